"""``bench.py --workload begupel``: prefill and decode of the Begupel family beside the closest other stack of the framework at equal size
(grouped-query attention, gated DeltaNet and a SwiGLU feed-forward for a parallel layer, gated DeltaNet for a lightning layer, bf16), and
each mixer, stream and element-wise kernel beside its counterpart with the share of its roofline that both reach.

Synthetic seeded token ids, random-init weights.  Device-timed with CUDA events; kernels are timed over a rotation of input sets
larger than L2 together.  Roofline of a kernel: the slower of its algorithmic bytes over the measured copy bandwidth and its products
over the measured bf16 GEMM rate."""
from __future__ import annotations

import torch

from ..config import LAYER_ATTENTION, LAYER_GDN, LAYER_MLP, AttentionConfig, ChannelDeltaConfig, GdnConfig, ModelConfig, begupel_config
from .dimesun import _graph_time, _meta, _time, peaks

SIZES = {"hidden": 2048, "heads": 16, "inter": 6144, "vocab": 32768, "window": 1024}


def counterpart_config(layers: int, **over) -> ModelConfig:
    """The attention / GDN hybrid with the same mixers per layer pair, width, heads, feed-forwards and vocabulary: attention without a
    feed-forward and GDN with one for a parallel layer, GDN without one for a lightning layer."""
    s, types, mlps = SIZES, [], []
    for i in range(layers):
        types += [LAYER_ATTENTION, LAYER_GDN] if i % 2 == 0 else [LAYER_GDN]
        mlps += ["none", LAYER_MLP] if i % 2 == 0 else ["none"]
    base = dict(model_type="nemotron_h_hybrid", vocab_size=s["vocab"], hidden_size=s["hidden"], intermediate_size=s["inter"],
                num_hidden_layers=len(types), num_attention_heads=s["heads"], num_key_value_heads=s["heads"] // 4, head_dim=128, rms_norm_eps=1e-6,
                rope_theta=1e6, layer_types=types, mlp_types=mlps, hidden_act="silu", gdn=GdnConfig(s["heads"], s["heads"], 128, 128, 4))
    base.update(over)
    return ModelConfig(**base)


def kernel_pairs(device) -> list:
    """One row per kernel or kernel group: time, roofline and the counterpart's."""
    from ..ops import Bigram, cuda as cu
    bw, fl = peaks()
    s, dt, n, d = SIZES, torch.bfloat16, SIZES["heads"], 128
    kvh, rows, h = n // 4, [], SIZES["hidden"]
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
        st = [torch.zeros(b, n, d, d, device=device) for _ in range(sets)]
        # ---- lightning attention beside the matrix-memory LSTM ----
        qkvg = [rnd(t, 4 * n * d).to(dt) for _ in range(sets)]
        gates, ns, nw = [rnd(t, 2 * n) * 2 for _ in range(sets)], [torch.zeros(b, n, d + 1, device=device) for _ in range(sets)], torch.ones(n * d, device=device)
        powers = ((1 - 2.0 ** -(2 + torch.arange(n, device=device, dtype=torch.float64) * 0.4))[:, None] ** torch.arange(257, device=device)).float()
        flops = 2.0 * t * n * (128 * d * 2 + 2 * d * d) if not decode else 0.0
        us = timer(lambda i: cu.lightning(qkvg[i], nw, powers, st[i], meta))
        us_mlstm = timer(lambda i: cu.mlstm(qkvg[i], gates[i], nw, st[i], ns[i], meta, d ** -0.5, 15.0, 1e-6, d))
        add(f"lightning attention (silu, recurrence, gate), {label}", us, 5 * io + state, flops, "mLSTM with head norm and gate", us_mlstm, 5 * io + state, flops)
        del gates, ns
        # ---- delta rule with head decays beside the gated delta rule and the channel-decay form ----
        sp, sc = ChannelDeltaConfig(n, n, d, d, 4, 0, 0, head_decay=True, silu_gate=True), ChannelDeltaConfig(n, n, d, d, 4)
        small = [rnd(t, 2 * n) for _ in range(sets)]
        cs = [torch.zeros(b, 3 * n * d, 3, device=device, dtype=dt) for _ in range(sets)]
        cw, al, hb, dn = (rnd(3 * n * d, 4) * 0.3).to(dt), torch.zeros(n, device=device), torch.full((n,), -4.0, device=device), torch.ones(d, device=device)
        us = timer(lambda i: cu.channel_delta(qkvg[i][:, :3 * n * d], small[i][:, n:], qkvg[i][:, 3 * n * d:], small[i][:, :n], cw, al, hb, dn, cs[i], st[i],
                                              meta, sp, 1e-6))
        decay, cb = [rnd(t, n * d) for _ in range(sets)], torch.full((n * d,), -4.0, device=device)
        us_ch = timer(lambda i: cu.channel_delta(qkvg[i][:, :3 * n * d], decay[i], qkvg[i][:, 3 * n * d:], small[i][:, :n], cw, al, cb, dn, cs[i], st[i], meta,
                                                 sc, 1e-6))
        del decay
        qkv, z = [x[:, :3 * n * d].contiguous() for x in qkvg], [x[:, 3 * n * d:].contiguous() for x in qkvg]
        a, bb = [x[:, :n].to(dt) for x in small], [x[:, n:].to(dt) for x in small]
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
        fd = 2.0 * t * n * (64 * d * 3 + 3 * d * d) if not decode else 0.0
        conv = 2 * 3 * b * 3 * n * d * 2
        name = f"delta rule, head decays (convolutions, recurrence, norm, gate), {label}"
        add(name, us, 5 * io + state + conv, fd, "channel-decay delta rule", us_ch, 5 * io + 2 * io + state + conv, fd)
        add(name, us, 5 * io + state + conv, fd, "gated delta rule with convolution, norm and gate", us_gdn, 5 * io + state + conv, fd)
        add(name, us, 5 * io + state + conv, fd, "gated delta rule alone", us_core, 4 * io + state, fd)
        del qkvg, small, cs, qkv, z, a, bb, q, k, v, st
        # ---- attention: window, rotated values ----
        pages = int(meta.page_table.max()) + 1
        kv = [rnd(pages, 2, kvh, 64, d).to(dt) for _ in range(sets)]
        qq = [rnd(t, n, d).to(dt) for _ in range(sets)]
        w = s["window"]
        see = lambda win: sum(min(p0 + i + 1, win) for ql, p0 in zip(q_lens, past) for i in range(ql))
        span = lambda win: sum(min(p0 + ql, win - 1 + ql) for ql, p0 in zip(q_lens, past))
        length = max(max(x + y for x, y in zip(q_lens, past)), 8192)
        tab, buf = rnd(length, d), [torch.empty(t, 2 * n * d, device=device, dtype=dt) for _ in range(sets)]
        us = timer(lambda i: cu.paged_attention(qq[i], kv[i], meta, d ** -0.5, w, fp32_weights=True, back=(tab, 0.7), out=buf[i][:, :n * d]))
        us_fp = timer(lambda i: cu.paged_attention(qq[i], kv[i], meta, d ** -0.5, fp32_weights=True))
        us_pl = timer(lambda i: cu.paged_attention(qq[i], kv[i], meta, d ** -0.5))
        cost = lambda win: (2 * io + span(win) * kvh * d * 4, 4.0 * see(win) * n * d)
        add(f"attention, window {w}, rotated values, fp32 weights, {label}", us, *cost(w), "attention, fp32 weights", us_fp, *cost(1 << 30))
        add(f"attention, window {w}, rotated values, fp32 weights, {label}", us, *cost(w), "attention", us_pl, *cost(1 << 30))
        sa = AttentionConfig(n, kvh, d, d, d, 1e6, d ** -0.5, window=w, row_norm=True, interleaved=True, rotated_values=True)
        packed = [rnd(t, (n + 2 * kvh) * d).to(dt) for _ in range(sets)]
        qn, kn = torch.ones(n * d, device=device), torch.ones(kvh * d, device=device)
        us = timer(lambda i: cu.turned_kv_write(packed[i], kv[i], meta, tab, tab, qn, kn, sa, 1e-6))
        us_like = timer(lambda i: cu.rope_kv_write(packed[i], kv[i], meta, tab, n, kvh, d, gw, gw, 1e-6))
        pb = 2 * t * (n + 2 * kvh) * d * 2
        add(f"row norms, rotation of q, k and v, cache write, {label}", us, pb, 0.0, "q / k norm, rotation, cache write", us_like, pb, 0.0)
        del kv, qq, packed, buf
        # ---- stream and feed-forward element-wise steps ----
        x, y, res = [rnd(t, h) for _ in range(sets)], [rnd(t, h).to(dt) for _ in range(sets)], [rnd(t, h).to(dt) for _ in range(sets)]
        ww, wb, alpha = torch.ones(h, device=device), torch.ones(h, device=device, dtype=dt), torch.ones((), device=device)
        taps, hist, sums = rnd(4, h) * 0.2, [torch.zeros(b, 3, h, device=device) for _ in range(sets)], [rnd(t, n * d // 32).abs() for _ in range(sets)]
        post = lambda i, **kw: cu.stream_post(x[i], y[i], ww, 4, 1e-6, meta, dt, None, None, None, kw.get("conv"), kw.get("history"), kw.get("out_norm"),
                                              kw.get("sums"))
        us_tanh = timer(lambda i: cu.stream_norm(x[i], ww, 1e-6, y[i], None, 1.0, None, 0.0, None, None, dt, alpha, ww))
        us_add = timer(lambda i: cu.add_rmsnorm(y[i], res[i], wb, 1e-6))
        row = t * h * (4 + 4 + 2 + 2)
        hb_ = 2 * b * 3 * h * 4
        for nm, u, by in (("output norm in parts + stream update (fp32)", timer(post), row),
                          ("output norm in parts + stream update (fp32) + input convolution", timer(lambda i: post(i, conv=taps, history=hist[i])), row + hb_),
                          ("the same behind lightning attention", timer(lambda i: post(i, conv=taps, history=hist[i], sums=(sums[i], n * d))), row + hb_ + t * n * d // 8)):
            add(f"{nm}, {label}", u, by, 0.0, "stream update (fp32) + tanh norm", us_tanh, row, 0.0)
            add(f"{nm}, {label}", u, by, 0.0, "residual (16-bit) + RMS norm", us_add, t * h * 8, 0.0)
        ids, table, big = torch.randint(0, 32768, (t,), device=device, dtype=torch.int32), rnd(32768, h).to(dt), rnd(65537, h).to(dt)
        bg = Bigram(big, torch.zeros(b, 1, dtype=torch.int32, device=device), 65536, 1000003, 8191)
        us = timer(lambda i: cu.stream_post(None, None, None, 4, 1e-6, meta, dt, ids, table, bg, taps, hist[i], None))
        us_like = timer(lambda i: cu.stream_norm(None, ww, 1e-6, None, None, 1.0, None, 0.0, ids, table, dt))
        add(f"embedding + bigram + input convolution, {label}", us, t * h * (2 + 2 + 4 + 2) + hb_, 0.0, "embedding + norm", us_like, t * h * (2 + 4 + 2), 0.0)
        gu = [rnd(t, 2 * s["inter"]).to(dt) for _ in range(sets)]
        us, us_like = timer(lambda i: cu.reglu(gu[i])), timer(lambda i: cu.swiglu(gu[i]))
        add(f"relu gate, {label}", us, t * s["inter"] * 6, 0.0, "silu gate", us_like, t * s["inter"] * 6, 0.0)
        del x, y, res, gu, table, big
    return rows


def model_pair(layers: int, device, args) -> dict:
    """Prefill and decode throughput of both stacks at a few shapes."""
    from ..runtime.llm import LLM
    from .workloads import _generate_timed
    s, out = SIZES, {}
    for name, cfg in (("begupel", begupel_config(layers, s["hidden"], s["vocab"], s["heads"], s["inter"], s["window"])),
                      ("attention / gdn hybrid", counterpart_config(layers))):
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
    first = models["begupel"]["batch 64, prompt 512"]
    return {"metric": "decode tok/s, Begupel at production-like layer sizes (bf16), beside a like-sized attention / GDN hybrid",
            "value": first["decode_tok_s"], "unit": "tok/s", "n_gpus": 1, "ms_per_step": first["decode_ms_per_step"],
            "config": {"layers": layers, **SIZES, "head_dim": 128, "l2": "kernel inputs rotate over sets larger than L2; weights exceed L2"},
            "models": models, "kernels": rows, "gpu_launches": int(cu.LAUNCHES - l0), "data": "synthetic (seeded token ids, random-init weights)",
            "dtype": "bf16"}
