"""``bench.py --workload debonex``: prefill and decode of the Debonex family beside the closest other stack of the framework at equal size
(gated DeltaNet for the channel-decay delta rule, grouped-query attention for latent and unit-norm attention, SwiGLU feed-forwards of
the same size, bf16), and each mixer, norm and feed-forward step beside its counterpart with the share of its roofline that both reach.

Synthetic seeded token ids, random-init weights.  Device-timed with CUDA events; kernels are timed over a rotation of input sets
larger than L2 together.  Roofline of a kernel: the slower of its algorithmic bytes over the measured copy bandwidth and its products
over the measured bf16 GEMM rate."""
from __future__ import annotations

import torch

from ..config import LAYER_ATTENTION, LAYER_GDN, LAYER_MLP, ChannelDeltaConfig, GdnConfig, LatentConfig, ModelConfig, debonex_config
from .dimesun import _graph_time, _meta, _time, peaks

SIZES = {"hidden": 2048, "heads": 16, "inter": 6144, "rank": 512, "vocab": 32768}


def counterpart_config(layers: int, **over) -> ModelConfig:
    """The GDN / attention hybrid of the same depth, width, heads, feed-forwards and vocabulary."""
    s = SIZES
    types = [LAYER_ATTENTION if i % 2 else LAYER_GDN for i in range(layers)]
    base = dict(model_type="nemotron_h_hybrid", vocab_size=s["vocab"], hidden_size=s["hidden"], intermediate_size=s["inter"],
                num_hidden_layers=layers, num_attention_heads=s["heads"], num_key_value_heads=s["heads"] // 4, head_dim=128, rms_norm_eps=1e-6,
                rope_theta=1e6, layer_types=types, mlp_types=[LAYER_MLP] * layers, hidden_act="silu", gdn=GdnConfig(s["heads"], s["heads"], 128, 128, 4))
    base.update(over)
    return ModelConfig(**base)


def kernel_pairs(device) -> list:
    """One row per kernel or kernel group: time, roofline and the counterpart's."""
    from ..ops import cuda as cu
    bw, fl = peaks()
    s, dt, n, d = SIZES, torch.bfloat16, SIZES["heads"], 128
    kvh, rows = n // 4, []
    rnd = lambda *shape: torch.randn(*shape, device=device, dtype=torch.float32)

    def add(name, us, bytes_, flops, like, like_us, like_bytes, like_flops):
        roof, lroof = (max(b / bw, f / fl) * 1e6 for b, f in ((bytes_, flops), (like_bytes, like_flops)))
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "share": round(roof / us, 4), "like": like,
                     "like_us": round(like_us, 2), "like_roofline_us": round(lroof, 2), "like_share": round(lroof / like_us, 4),
                     "distance_ratio": round((us / roof) / (like_us / lroof), 3)})

    for label, q_lens, past in (("prefill 8x1024", [1024] * 8, [0] * 8), ("prefill 1x8192", [8192], [0]), ("decode b64", [1] * 64, [1535] * 64),
                                ("decode b8", [1] * 8, [1535] * 8), ("decode b1", [1], [8191])):
        t, b = sum(q_lens), len(q_lens)
        decode = max(q_lens) == 1
        meta = _meta(q_lens, past, device)
        sets = 3 if not decode else max(2, min(8, 512 // b))
        timer = (lambda fn, k=sets: _graph_time(fn, k)) if decode else (lambda fn, k=sets: _time(lambda i: fn(i % k), 3 * k))
        io = t * n * d * 2
        state = b * n * d * d * 4 * (2 if decode else 1)
        # ---- recurrent mixers: projections in, gated head outputs out ----
        sp = ChannelDeltaConfig(n, n, d, d, 4)
        qkv, gate = [rnd(t, 3 * n * d).to(dt) for _ in range(sets)], [rnd(t, n * d) if t <= 128 else rnd(t, n * d).to(dt) for _ in range(sets)]
        decay, beta = [rnd(t, n * d) for _ in range(sets)], [rnd(t, n) for _ in range(sets)]
        st = [torch.zeros(b, n, d, d, device=device) for _ in range(sets)]
        cs = [torch.zeros(b, 3 * n * d, 3, device=device, dtype=dt) for _ in range(sets)]
        cw, al, bias, nw = (rnd(3 * n * d, 4) * 0.3).to(dt), torch.zeros(n, device=device), torch.full((n * d,), -4.0, device=device), torch.ones(d, device=device)
        us = timer(lambda i: cu.channel_delta(qkv[i], decay[i], gate[i], beta[i], cw, al, bias, nw, cs[i], st[i], meta, sp, 1e-6))
        a, bb = [rnd(t, n).to(dt) for _ in range(sets)], [rnd(t, n).to(dt) for _ in range(sets)]
        z = [x.to(dt) for x in gate]
        gw, db = torch.ones(d, device=device, dtype=dt), torch.zeros(n, device=device)

        def gdn(i):                                    # as the gated-DeltaNet mixer runs it between its projections
            y = cu.causal_conv1d(qkv[i], cw, None, cs[i], meta)
            q, k, v = y.split([n * d] * 3, dim=-1)
            o = cu.gated_delta_rule(q.reshape(t, n, d), k.reshape(t, n, d), v.reshape(t, n, d), a[i], bb[i], al, db, st[i], meta)
            o = cu.rmsnorm(o.reshape(t * n, d), gw, 1e-6).reshape(t, n * d)
            zf = z[i].float()
            return (o.float() * (zf * torch.sigmoid(zf))).to(dt)
        us_gdn = timer(gdn)
        q, k, v = ([x[:, j * n * d:(j + 1) * n * d].reshape(t, n, d).contiguous() for x in qkv] for j in range(3))
        us_core = timer(lambda i: cu.gated_delta_rule(q[i], k[i], v[i], a[i], bb[i], al, db, st[i], meta))
        # chunked form, 64 rows: two score products, the solve applied to values, three products with the state
        flops = 2.0 * t * n * (64 * d * 3 + 3 * d * d) if not decode else 0.0
        conv = 2 * 3 * b * 3 * n * d * 2
        gb = gate[0].element_size() * gate[0].numel()
        add(f"channel delta (convolutions, recurrence, norm, gate), {label}", us, 4 * io + 2 * io + gb + state + conv, flops,
            "gated delta rule with convolution, norm and gate", us_gdn, 5 * io + state + conv, flops)
        add(f"channel delta (convolutions, recurrence, norm, gate), {label}", us, 4 * io + 2 * io + gb + state + conv, flops,
            "gated delta rule alone", us_core, 4 * io + state, flops)
        del qkv, gate, decay, beta, st, cs, a, bb, z, q, k, v
        # ---- attention ----
        vis = sum((2 * p0 + ql + 1) * ql // 2 for ql, p0 in zip(q_lens, past))
        total = sum(ql + p0 for ql, p0 in zip(q_lens, past))
        pages = int(meta.page_table.max()) + 1
        ls = LatentConfig(n, d, 64, d, s["rank"], 1e4, 192 ** -0.5)
        kv = [rnd(pages, 2, kvh, 64, d).to(dt) for _ in range(sets)]
        qq = [rnd(t, n, d).to(dt) for _ in range(sets)]
        us_gqa = timer(lambda i: cu.paged_attention(qq[i], kv[i], meta, d ** -0.5, fp32_weights=True))
        us_plain = timer(lambda i: cu.paged_attention(qq[i], kv[i], meta, d ** -0.5))
        kvb = (vis if decode else t) * kvh * d * 4
        temp = torch.ones(max(q_lens[0] + past[0], 8192), device=device)
        packed = [rnd(t, (n + 2 * kvh) * d).to(dt) for _ in range(sets)]
        cs_t = rnd(max(q_lens[0] + past[0], 8192), d)
        us_unit = timer(lambda i: cu.unit_kv_write(packed[i], kv[i], meta, temp, n, kvh, d, d, 1e-6))
        us_rope = timer(lambda i: cu.rope_kv_write(packed[i], kv[i], meta, cs_t, n, kvh, d, gw, gw, 1e-6))
        pb = 2 * t * (n + 2 * kvh) * d * 2
        add(f"unit norm, temperature, cache write, {label}", us_unit, pb, 0.0, "q / k norm, rotation, cache write", us_rope, pb, 0.0)
        add(f"attention with fp32 weights, {label}", us_gqa, 2 * io + kvb, 4.0 * vis * n * d, "attention", us_plain, 2 * io + kvb, 4.0 * vis * n * d)
        del kv, qq, packed
        row = ls.pad
        width = n * (ls.k_pad + ls.rot_pad) + row
        lat = [rnd(pages, 1, 1, 64, row).to(dt) for _ in range(sets)]
        x = [rnd(t, width).to(dt) for _ in range(sets)]
        ups = [(rnd(n * (ls.k_pad + ls.v_pad), ls.rank_pad) * 0.05).to(dt) for _ in range(2)]
        kts = [u[:n * ls.k_pad].view(n, ls.k_pad, ls.rank_pad).transpose(1, 2).contiguous() for u in ups]
        us = timer(lambda i: cu.latent_attention(x[i], lat[i], meta, ups[i % 2], kts[i % 2], ls))
        up_b = ups[0].numel() * 2
        lb = (total if decode else t) * row * 2
        up_f = 2.0 * (t if decode else total) * ups[0].numel()
        att_f = 2.0 * vis * n * (2 * ls.rank_pad + 64) if decode else 2.0 * vis * n * (d + 64 + d)
        add(f"latent attention with key / value expansion, {label}", us, t * n * (192 + d) * 2 + lb + up_b, up_f + att_f,
            "grouped-query attention, fp32 weights", us_gqa, 2 * io + kvb, 4.0 * vis * n * d)
        add(f"latent attention with key / value expansion, {label}", us, t * n * (192 + d) * 2 + lb + up_b, up_f + att_f,
            "grouped-query attention", us_plain, 2 * io + kvb, 4.0 * vis * n * d)
        cw_t = rnd(max(q_lens[0] + past[0], 8192), 64)
        nr = torch.ones(ls.rank_pad, device=device)
        us = timer(lambda i: cu.latent_write(x[i], lat[i], meta, cw_t, nr, ls, 1e-6))
        add(f"latent norm, rotation, cache write, {label}", us, 2 * t * (n * 64 + row) * 2, 0.0, "q / k norm, rotation, cache write", us_rope, pb, 0.0)
        del lat, x, ups, kts
        # ---- stream and feed-forward element-wise steps ----
        h = s["hidden"]
        stream, a2, res = [rnd(t, h) for _ in range(sets)], [rnd(t, h).to(dt) for _ in range(sets)], [rnd(t, h).to(dt) for _ in range(sets)]
        w, alpha, wb = torch.ones(h, device=device), torch.ones((), device=device), torch.ones(h, device=device, dtype=dt)
        us = timer(lambda i: cu.stream_norm(stream[i], w, 1e-6, a2[i], None, 1.0, None, 0.0, None, None, dt, alpha, w))
        us_like = timer(lambda i: cu.add_rmsnorm(a2[i], res[i], wb, 1e-6))
        add(f"stream update (fp32) + tanh norm, {label}", us, t * h * (4 + 4 + 2 + 2), 0.0, "residual (16-bit) + RMS norm", us_like, t * h * 8, 0.0)
        gu = [rnd(t, 2 * s["inter"]).to(dt) for _ in range(sets)]
        us, us_like = timer(lambda i: cu.geglu(gu[i])), timer(lambda i: cu.swiglu(gu[i]))
        add(f"gelu gate, {label}", us, t * s["inter"] * 6, 0.0, "silu gate", us_like, t * s["inter"] * 6, 0.0)
        del stream, a2, res, gu
    return rows


def model_pair(layers: int, device, args) -> dict:
    """Prefill and decode throughput of both stacks at a few shapes."""
    from ..runtime.llm import LLM
    from .workloads import _generate_timed
    s, out = SIZES, {}
    for name, cfg in (("debonex", debonex_config(layers, s["hidden"], s["vocab"], s["heads"], s["inter"], s["rank"])),
                      ("gdn hybrid", counterpart_config(layers))):
        llm = LLM(cfg, device=str(device), max_batch_size=64, max_input_len=8192, max_kv_cache_capacity=8192 + 128, max_num_tokens=4 * 8192,
                  kv_pages=(64 * 640) // 64 + 200, random_init_seed=0)
        g = torch.Generator().manual_seed(1234)
        res = {}
        for b, sl, ol in [(8, 1024, 65), (1, 8192, 65), (64, 512, 65)]:
            prompts = torch.randint(0, cfg.vocab_size, (b, sl), generator=g, dtype=torch.int32).to(device)
            pre, dec = _generate_timed(llm, prompts, ol, max(2, args.steps), max(3, args.warmup))
            res[f"batch {b}, prompt {sl}"] = {"prefill_ms": round(pre, 3), "prefill_tok_s": round(b * sl / pre * 1e3, 1),
                                              "decode_ms_per_step": round(dec / (ol - 1), 4), "decode_tok_s": round(b * (ol - 1) / dec * 1e3, 1)}
            for seat in range(b):
                llm.kv.free(seat)
        out[name] = res
        llm.close()
        del llm
        torch.cuda.empty_cache()
    return out


def run(args) -> dict:
    from ..ops import cuda as cu
    torch.cuda.set_device(0)
    dev = torch.device("cuda", 0)
    layers = args.layers or 12
    l0 = cu.LAUNCHES
    rows = kernel_pairs(dev)
    models = model_pair(layers, dev, args)
    cu.Workspace.get(dev).check_status()
    first = models["debonex"]["batch 64, prompt 512"]
    return {"metric": "decode tok/s, Debonex at production-like layer sizes (bf16), beside a like-sized GDN / attention hybrid",
            "value": first["decode_tok_s"], "unit": "tok/s", "n_gpus": 1, "ms_per_step": first["decode_ms_per_step"],
            "config": {"layers": layers, **SIZES, "head_dim": 128, "l2": "kernel inputs rotate over sets larger than L2; weights exceed L2"},
            "models": models, "kernels": rows, "gpu_launches": int(cu.LAUNCHES - l0), "data": "synthetic (seeded token ids, random-init weights)",
            "dtype": "bf16"}
