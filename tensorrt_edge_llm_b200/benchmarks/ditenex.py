"""``bench.py --workload ditenex``: prefill and decode of the Ditenex family beside the closest other stack of the framework at equal size
(windowed grouped-query attention with q / k norms and rotary positions, SwiGLU feed-forwards and softmax-top-k experts with a shared one
in turn, bf16), and each attention, stream, activation and expert kernel beside its counterpart with the share of its roofline
that both reach.

Synthetic seeded token ids, random-init weights.  Device-timed with CUDA events; kernels are timed over a rotation of input sets
larger than L2 together.  Roofline of a kernel: the slower of its algorithmic bytes over the measured copy bandwidth and its products
over the measured bf16 GEMM rate."""
from __future__ import annotations

import torch

from ..config import LAYER_ATTENTION, LAYER_MLP, LAYER_MOE, AttentionConfig, ModelConfig, ditenex_config
from .dimesun import _graph_time, _meta, _time, peaks

SIZES = {"hidden": 2048, "heads": 16, "inter": 6144, "experts": 64, "top_k": 4, "expert_inter": 768, "vocab": 32768, "window": 1024}


def _config(layers: int, **over) -> ModelConfig:
    s = SIZES
    return ditenex_config(layers, s["hidden"], s["vocab"], s["heads"], s["inter"], s["experts"], s["top_k"], s["expert_inter"], s["window"], **over)


def counterpart_config(layers: int, **over) -> ModelConfig:
    """Attention with the same heads and window; dense and expert feed-forwards of the same sizes in turn (a gated unit in place of the
    un-gated one has half as much again to compute: its inner size is two thirds)."""
    s = SIZES
    base = dict(model_type="nemotron_h_hybrid", vocab_size=s["vocab"], hidden_size=s["hidden"], intermediate_size=s["inter"] * 2 // 3, num_hidden_layers=layers,
                num_attention_heads=s["heads"], num_key_value_heads=s["heads"] // 4, head_dim=128, rms_norm_eps=1e-6, rope_theta=1e6, has_qk_norm=True,
                sliding_window=s["window"], layer_types=[LAYER_ATTENTION] * layers, mlp_types=[LAYER_MOE if i % 2 else LAYER_MLP for i in range(layers)],
                hidden_act="silu", num_experts=s["experts"], num_experts_per_tok=s["top_k"], moe_intermediate_size=s["expert_inter"],
                shared_expert_intermediate_size=s["expert_inter"], max_position_embeddings=16384)
    base.update(over)
    return ModelConfig(**base)


def kernel_pairs(device) -> list:
    """One row per kernel or kernel group: time, roofline and the counterpart's."""
    from ..models.qwen3_moe import MoEBlock, SharedExpertsBlock
    from ..ops import cuda as cu
    bw, fl = peaks()
    s, dt, n, d = SIZES, torch.bfloat16, SIZES["heads"], 128
    kvh, rows, h, w = n // 4, [], SIZES["hidden"], SIZES["window"]
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
        # ---- attention ----
        pages = int(meta.page_table.max()) + 1
        kv = [rnd(pages, 2, kvh, 64, d).to(dt) for _ in range(sets)]
        see = sum(min(p0 + i + 1, w) for ql, p0 in zip(q_lens, past) for i in range(ql))
        span = sum(min(p0 + ql, w - 1 + ql) for ql, p0 in zip(q_lens, past))
        sp = AttentionConfig(n, kvh, d, d, 0, scale=d ** -0.5, fp32_weights=True, window=w, mixed_scores=True, distance_bias=True, value_mix=True, qkv_bias=True,
                             out_gate=True)
        packed, first = [rnd(t, (2 * n + 2 * kvh) * d).to(dt) for _ in range(sets)], [rnd(t, kvh * d).to(dt) for _ in range(sets)]
        mix, share = torch.eye(n, device=device) + 0.2 * rnd(n, n), torch.tensor(0.4, device=device)
        slopes = 2.0 ** (-8.0 * (torch.arange(n, device=device) + 1) / n)
        g0, qkv = (n + 2 * kvh) * d, [x[:, :(n + 2 * kvh) * d].contiguous() for x in packed]
        tab, gw = rnd(max(8192, *(x + y for x, y in zip(q_lens, past))), d), torch.ones(d, device=device, dtype=dt)
        write = lambda i: cu.mixed_kv_write(packed[i], kv[i], meta, mix, first[i], share, sp)
        wide = [write(i) for i in range(sets)]
        attend = lambda i: cu.mixed_attention(wide[i], kv[i], meta, slopes, packed[i][:, g0:], sp)
        rope = lambda i: cu.rope_kv_write(qkv[i], kv[i], meta, tab, n, kvh, d, gw, gw, 1e-6)
        qq = [rope(i) for i in range(sets)]
        fp32w = lambda i: cu.paged_attention(qq[i], kv[i], meta, d ** -0.5, w, fp32_weights=True)
        plain = lambda i: cu.paged_attention(qq[i], kv[i], meta, d ** -0.5, w)
        us_w, us_a, us_r, us_f, us_p = (timer(f) for f in (write, attend, rope, fp32w, plain))
        us_both = timer(lambda i: cu.mixed_attention(write(i), kv[i], meta, slopes, packed[i][:, g0:], sp))
        us_like = timer(lambda i: cu.paged_attention(rope(i), kv[i], meta, d ** -0.5, w, fp32_weights=True))
        wb = wide[0].numel() * 2
        ab, af = span * kvh * d * 4, 4.0 * see * n * d
        pb = 2 * t * (n + 2 * kvh) * d * 2
        add(f"mixed attention (wide queries), window {w}, gate, {label}", us_a, wb + 2 * io + ab, af + 2.0 * see * n * n, "attention, same window, fp32 weights", us_f,
            2 * io + ab, af)
        add(f"mixed attention (wide queries), window {w}, gate, {label}", us_a, wb + 2 * io + ab, af + 2.0 * see * n * n, "attention, same window", us_p, 2 * io + ab, af)
        add(f"wide queries, mixed values, cache write, {label}", us_w, pb - io + wb + t * kvh * d * 2, 0.0, "q / k norm, rotation, cache write", us_r, pb, 0.0)
        add(f"the two together, {label}", us_both, pb + ab + 2 * io + t * kvh * d * 2, af + 2.0 * see * n * n,
            "q / k norm, rotation, cache write + attention, fp32 weights", us_like, pb + ab + io, af)
        del kv, packed, first, qkv, wide, qq
        # ---- stream ----
        x, y, res = [rnd(t, h) for _ in range(sets)], [rnd(t, h).to(dt) for _ in range(sets)], [rnd(t, h).to(dt) for _ in range(sets)]
        ww, wb16, alpha, amount = torch.ones(h, device=device), torch.ones(h, device=device, dtype=dt), torch.ones((), device=device), torch.rand(h, device=device)
        state = [torch.zeros(b, 1, h, device=device) for _ in range(sets)]
        step = lambda i, **kw: cu.stream_sandwich(x[i], 1e-6, meta, dt, None, None, None, y[i], kw.get("routed"), ww, 0.5, ww, kw.get("shift"), kw.get("state"))
        us_tanh = timer(lambda i: cu.stream_norm(x[i], ww, 1e-6, y[i], None, 1.0, None, 0.0, None, None, dt, alpha, ww))
        us_post = timer(lambda i: cu.stream_post(x[i], y[i], ww, 1, 1e-6, meta, dt, None, None, None, None, None, None))
        us_add = timer(lambda i: cu.add_rmsnorm(y[i], res[i], wb16, 1e-6))
        row = t * h * (4 + 4 + 2 + 2)
        for nm, u, by in (("norm, stream update (fp32), norm", timer(step), row),
                          ("norm, stream update (fp32), norm, token shift", timer(lambda i: step(i, shift=amount, state=state[i])), row + 2 * b * h * 4)):
            add(f"{nm}, {label}", u, by, 0.0, "stream update (fp32) + tanh norm", us_tanh, row, 0.0)
            add(f"{nm}, {label}", u, by, 0.0, "norm + stream update (fp32)", us_post, row, 0.0)
            add(f"{nm}, {label}", u, by, 0.0, "residual (16-bit) + RMS norm", us_add, t * h * 8, 0.0)
        ids, table, pos = torch.randint(0, 32768, (t,), device=device, dtype=torch.int32), rnd(32768, h).to(dt), rnd(8192, h).to(dt)
        us = timer(lambda i: cu.stream_sandwich(None, 1e-6, meta, dt, ids, table, pos, None, None, None, 1.0, ww, amount, state[i]))
        us_like = timer(lambda i: cu.stream_norm(None, ww, 1e-6, None, None, 1.0, None, 0.0, ids, table, dt))
        add(f"embedding + position, norm, token shift, {label}", us, t * h * (2 + 2 + 4 + 2) + 2 * b * h * 4, 0.0, "embedding + norm", us_like, t * h * (2 + 4 + 2), 0.0)
        # ---- activation ----
        up, gu, coef = [rnd(t, s["inter"]).to(dt) for _ in range(sets)], [rnd(t, 2 * s["inter"]).to(dt) for _ in range(sets)], torch.tensor([1.0, 1.2], device=device)
        us, us_sq, us_sw = timer(lambda i: cu.xielu(up[i], coef)), timer(lambda i: cu.relu2(up[i])), timer(lambda i: cu.swiglu(gu[i]))
        add(f"xIELU, {label}", us, t * s["inter"] * 4, 0.0, "squared relu", us_sq, t * s["inter"] * 4, 0.0)
        add(f"xIELU, {label}", us, t * s["inter"] * 4, 0.0, "silu gate", us_sw, t * s["inter"] * 6, 0.0)
        del up, gu, res, table, pos
        # ---- experts with router, shared expert and stream update ----
        cfg, qcfg = _config(2), counterpart_config(2)
        gen = torch.Generator().manual_seed(0)
        with torch.device(device):
            ours = [SharedExpertsBlock(cfg, cfg.layer_specs[1].moe, "m") for _ in range(2)]
            theirs = [MoEBlock(qcfg, "m") for _ in range(2)]
        for m in ours + theirs:
            for lin in m.modules():
                if hasattr(lin, "weight") and lin.weight is not None and lin.weight.dim() == 2:
                    lin.weight.data.normal_(0.0, 0.02)
        for m in [o.routed for o in ours] + theirs:
            m.random_init(gen)
        two = (lambda fn: _graph_time(fn, 2)) if decode else (lambda fn: _time(lambda i: fn(i % 2), 10))

        def block(i):
            shared, routed = ours[i](y[i])
            return cu.stream_sandwich(x[i], 1e-6, meta, dt, None, None, None, shared, routed, ww, 0.5, ww, amount, state[i])

        def like(i):
            return cu.add_rmsnorm(theirs[i](y[i]), y[i], wb16, 1e-6)
        hit = min(s["experts"], t * s["top_k"])
        eb, ef = (hit + 1) * 3 * h * s["expert_inter"] * 2, 6.0 * t * (s["top_k"] + 1) * h * s["expert_inter"]
        add(f"experts with router and shared expert + stream update + norm, {label}", two(block), eb + 8 * t * h * 2, ef,
            "softmax-top-k experts with shared expert + add + norm", two(like), eb + 6 * t * h * 2, ef)
        del ours, theirs, x, y
    return rows


def model_pair(layers: int, device, args) -> dict:
    """Prefill and decode throughput of both stacks at a few shapes."""
    from ..runtime.llm import LLM
    from .workloads import _generate_timed
    out = {}
    for name, cfg in (("ditenex", _config(layers)), ("windowed attention, dense / experts", counterpart_config(layers))):
        llm = LLM(cfg, device=str(device), max_batch_size=64, max_input_len=8192, max_kv_cache_capacity=8192 + 128, max_num_tokens=4 * 8192,
                  kv_pages=(64 * 640) // 64 + 200, random_init_seed=0)
        llm.kv.bounded_swa = False                       # both keep their pages, both decode from captured steps
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
    first = models["ditenex"]["batch 64, prompt 512"]
    return {"metric": "decode tok/s, Ditenex at production-like layer sizes (bf16), beside a like-sized windowed attention / experts stack",
            "value": first["decode_tok_s"], "unit": "tok/s", "n_gpus": 1, "ms_per_step": first["decode_ms_per_step"],
            "config": {"layers": layers, **SIZES, "head_dim": 128, "l2": "kernel inputs rotate over sets larger than L2; weights exceed L2"},
            "models": models, "kernels": rows, "gpu_launches": int(cu.LAUNCHES - l0), "data": "synthetic (seeded token ids, random-init weights)",
            "dtype": "bf16"}
