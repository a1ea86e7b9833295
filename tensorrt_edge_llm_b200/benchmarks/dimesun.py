"""``bench.py --workload dimesun``: prefill and decode of the Dimesun family beside the closest other stack of the framework at equal
size (gated DeltaNet in place of mLSTM, full attention in place of chunked, softmax-top-k SwiGLU experts of the same sizes, bf16), and
each recurrent, attention, expert and stream kernel beside its counterpart with the share of its roofline that both reach.

Synthetic seeded token ids, random-init weights.  Device-timed with CUDA events; kernels are timed over a rotation of input sets
larger than L2 together.  Roofline of a kernel: the slower of its algorithmic bytes over the measured copy bandwidth and its products
over the measured bf16 GEMM rate."""
from __future__ import annotations

import json
import os

import torch

from ..config import LAYER_ATTENTION, LAYER_GDN, LAYER_MOE, GdnConfig, ModelConfig, dimesun_config

SIZES = {"hidden": 2048, "heads": 16, "experts": 64, "top_k": 4, "inter": 768, "vocab": 32768, "chunk": 2048}


def counterpart_config(layers: int, **over) -> ModelConfig:
    """The GDN / attention / MoE hybrid of the same depth, width, heads, experts and vocabulary."""
    s = SIZES
    types = [LAYER_ATTENTION if i % 3 == 2 else LAYER_GDN for i in range(layers)]
    base = dict(model_type="nemotron_h_hybrid", vocab_size=s["vocab"], hidden_size=s["hidden"], intermediate_size=4 * s["hidden"],
                num_hidden_layers=layers, num_attention_heads=s["heads"], num_key_value_heads=s["heads"] // 4, head_dim=128, rms_norm_eps=1e-6,
                rope_theta=1e6, layer_types=types, mlp_types=[LAYER_MOE] * layers, num_experts=s["experts"], num_experts_per_tok=s["top_k"],
                moe_intermediate_size=s["inter"], gdn=GdnConfig(s["heads"], s["heads"], 128, 128, 4))
    base.update(over)
    return ModelConfig(**base)


def peaks() -> tuple:
    """(bytes/s, FLOP/s) measured on this part, or the fallback figures."""
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path, "r", encoding="utf-8") as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12
    return 6650e9, 1590e12


def _time(fn, iters: int, warm: int = 3) -> float:
    """Microseconds per call of ``fn(i)``; ``i`` rotates the inputs."""
    for i in range(warm):
        fn(i)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for i in range(iters):
        fn(i)
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e3 / iters


def _graph_time(fn, sets: int, iters: int = 20) -> float:
    """Microseconds per call with the launches of one rotation captured in a graph (decode sizes: no host time between kernels)."""
    for i in range(sets):
        fn(i)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(sets):
            fn(i)
    return _time(lambda _: g.replay(), iters) / sets


def _meta(q_lens, past, device):
    from ..ops.meta import build_step_meta
    pages = max((q + p + 63) // 64 for q, p in zip(q_lens, past))
    table = torch.arange(len(q_lens) * pages, dtype=torch.int32).reshape(len(q_lens), pages)
    return build_step_meta(q_lens, past, table, 64, device=device)


def kernel_pairs(device) -> list:
    """One row per kernel or kernel group: time, roofline and the counterpart's."""
    from ..config import MoeConfig, qwen3_30b_a3b_config
    from ..models.qwen3_moe import GatedExperts, MoEBlock
    from ..ops import cuda as cu
    bw, fl = peaks()
    s, dt, n, d = SIZES, torch.bfloat16, SIZES["heads"], 128
    kvh = n // 4
    rows = []
    rnd = lambda *shape: torch.randn(*shape, device=device, dtype=torch.float32)

    def add(name, us, bytes_, flops, like, like_us, like_bytes, like_flops):
        roof, lroof = (max(b / bw, f / fl) * 1e6 for b, f in ((bytes_, flops), (like_bytes, like_flops)))
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "share": round(roof / us, 4), "like": like,
                     "like_us": round(like_us, 2), "like_roofline_us": round(lroof, 2), "like_share": round(lroof / like_us, 4),
                     "distance_ratio": round((us / roof) / (like_us / lroof), 3)})

    for label, q_lens, past in (("prefill 8x1024", [1024] * 8, [0] * 8), ("prefill 1x8192", [8192], [0]), ("decode b64", [1] * 64, [1535] * 64),
                                ("decode b8", [1] * 8, [1535] * 8)):
        t, b = sum(q_lens), len(q_lens)
        decode = max(q_lens) == 1
        meta = _meta(q_lens, past, device)
        sets = 3 if not decode else max(2, min(8, 512 // b))
        timer = (lambda fn, k=sets: _graph_time(fn, k)) if decode else (lambda fn, k=sets: _time(lambda i: fn(i % k), 3 * k))
        # ---- recurrent mixers: rows in, state read and written once, rows out ----
        qkvg = [rnd(t, 4 * n * d).to(dt) for _ in range(sets)]
        gates = [rnd(t, 2 * n) * 2 for _ in range(sets)]
        st = [torch.zeros(b, n, d, d, device=device) for _ in range(sets)]
        ns = [torch.zeros(b, n, d + 1, device=device) for _ in range(sets)]
        nw = torch.ones(n * d, device=device)
        us = timer(lambda i: cu.mlstm(qkvg[i], gates[i], nw, st[i], ns[i], meta, d ** -0.5, 15.0, 1e-6, d))
        state = b * n * d * d * 4 * (2 if decode else 1)
        flops = 2.0 * t * n * (128 * d * 2 + 2 * d * d) if not decode else 0.0
        qkv = [x[:, :3 * n * d].contiguous() for x in qkvg]
        q, k, v = ([x[:, j * n * d:(j + 1) * n * d].reshape(t, n, d).contiguous() for x in qkv] for j in range(3))
        a, bb = [rnd(t, n).to(dt) for _ in range(sets)], [rnd(t, n).to(dt) for _ in range(sets)]
        al, db = torch.zeros(n, device=device), torch.zeros(n, device=device)
        z = [x[:, 3 * n * d:].contiguous() for x in qkvg]
        gw = torch.ones(d, device=device, dtype=dt)

        def gdn(i):                                    # with the norm and gate that follow it, as the mixer runs them
            o = cu.gated_delta_rule(q[i], k[i], v[i], a[i], bb[i], al, db, st[i], meta)
            o = cu.rmsnorm(o.reshape(t * n, d), gw, 1e-6).reshape(t, n * d)
            zf = z[i].float()
            return (o.float() * (zf * torch.sigmoid(zf))).to(dt)
        us_core = timer(lambda i: cu.gated_delta_rule(q[i], k[i], v[i], a[i], bb[i], al, db, st[i], meta))
        us_gdn = timer(gdn)
        io = t * n * d * 2
        gflops = 2.0 * t * n * (64 * d * 3 + 3 * d * d) if not decode else 0.0
        add(f"mlstm (recurrence, head norm, gate), {label}", us, 5 * io + gates[0].numel() * 4 + state, flops,
            "gated delta rule, norm and gate", us_gdn, 5 * io + state, gflops)
        add(f"mlstm (recurrence, head norm, gate), {label}", us, 5 * io + gates[0].numel() * 4 + state, flops,
            "gated delta rule alone", us_core, 4 * io + state, gflops)
        del qkvg, gates, st, ns, qkv, q, k, v, a, bb, z
        # ---- attention: chunked with a zero sink against full causal ----
        pages = int(meta.page_table.max()) + 1
        kv = [rnd(pages, 2, kvh, 64, d).to(dt) for _ in range(sets)]
        qq = [rnd(t, n, d).to(dt) for _ in range(sets)]
        sinks = torch.zeros(n, device=device)
        for chunk in (s["chunk"], 512):
            # the counterpart sees as many keys: plain causal attention over the same rows cut into sequences of one chunk each
            vis = sum((p % chunk) + 1 for ql, p0 in zip(q_lens, past) for p in range(p0, p0 + ql))
            cut = [(min(chunk, ql - c), p0 % chunk) for ql, p0 in zip(q_lens, past) for c in range(0, ql, chunk)]
            like = _meta([c for c, _ in cut], [p for _, p in cut], device)
            us = timer(lambda i: cu.paged_attention(qq[i], kv[i], meta, d ** -0.5, None, sinks, chunk=chunk, fp32_weights=True))
            us_like = timer(lambda i: cu.paged_attention(qq[i], kv[i], like, d ** -0.5, None, None))
            kvb = (vis if decode else t) * kvh * d * 4
            add(f"chunked attention (chunk {chunk}, sink, fp32 weights), {label}", us, 2 * io + kvb, 4.0 * vis * n * d,
                f"causal attention, {len(cut)} sequences of the chunk", us_like, 2 * io + kvb, 4.0 * vis * n * d)
        del kv, qq
        # ---- experts, the stream kernel, the fp32-output product ----
        cfg = dimesun_config(3, s["hidden"], s["vocab"], n, s["experts"], s["top_k"], s["inter"], s["chunk"])
        qcfg = qwen3_30b_a3b_config(hidden_size=s["hidden"], num_experts=s["experts"], num_experts_per_tok=s["top_k"], moe_intermediate_size=s["inter"],
                                    num_hidden_layers=1)
        gen = torch.Generator().manual_seed(0)
        with torch.device(device):
            ours = [GatedExperts(cfg, MoeConfig(s["experts"], s["top_k"], s["inter"], 7.0), "m") for _ in range(2)]
            theirs = [MoEBlock(qcfg, "m") for _ in range(2)]
        for m in ours + theirs:
            m.random_init(gen)
        x = [rnd(t, s["hidden"]).to(dt) for _ in range(2)]
        rw, rb = rnd(s["experts"], s["hidden"]).to(dt), rnd(s["experts"])
        stream = rnd(t, s["hidden"])
        w = torch.zeros(s["hidden"], device=device)
        two = (lambda fn: _graph_time(fn, 2)) if decode else (lambda fn: _time(lambda i: fn(i % 2), 10))

        def block(i):
            r = ours[i](x[i], cu.gemm_f32out(x[i], rw, rb))
            return cu.stream_norm(stream, w, 1e-6, x[i], r, 0.5, None, 1.0, None, None, dt)

        def like(i):
            y = theirs[i](x[i])
            return cu.add_rmsnorm(y, x[i], theirs[i].gate.weight[0], 1e-6)
        hit = min(s["experts"], t * s["top_k"])
        wb, mf = hit * 3 * s["hidden"] * s["inter"] * 2, 6.0 * t * s["top_k"] * s["hidden"] * s["inter"]
        hb = t * s["hidden"] * 2
        add(f"experts (with router) + stream update + norm, {label}", two(block), wb + 8 * hb, mf, "Qwen3-style experts (with router) + add + norm", two(like), wb + 6 * hb, mf)
        del ours, theirs, x
    return rows


def model_pair(layers: int, device, args) -> dict:
    """Prefill and decode throughput of both stacks at a few shapes."""
    from ..runtime.llm import LLM
    from .workloads import _generate_timed
    s, out = SIZES, {}
    shapes = [(8, 1024, 65), (1, 8192, 65), (64, 512, 65)]
    for name, cfg in (("dimesun", dimesun_config(layers, s["hidden"], s["vocab"], s["heads"], s["experts"], s["top_k"], s["inter"], s["chunk"])),
                      ("dimesun, middle third looped twice", dimesun_config(layers, s["hidden"], s["vocab"], s["heads"], s["experts"], s["top_k"],
                                                                            s["inter"], s["chunk"], loop_start=layers // 3,
                                                                            loop_stop=2 * layers // 3, loop_times=2)),
                      ("gdn hybrid", counterpart_config(layers))):
        if cfg.loop_stop:
            runs = [cfg.layer_specs[i] for i in cfg.layer_run_ids]
            cfg.num_hidden_layers, cfg.layer_types, cfg.mlp_types = len(runs), [r.kind for r in runs], [LAYER_MOE] * len(runs)
        llm = LLM(cfg, device=str(device), max_batch_size=64, max_input_len=8192, max_kv_cache_capacity=8192 + 128, max_num_tokens=4 * 8192,
                  kv_pages=(64 * 640) // 64 + 200, random_init_seed=0)
        g = torch.Generator().manual_seed(1234)
        res = {}
        for b, sl, ol in shapes:
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
    first = models["dimesun"]["batch 64, prompt 512"]
    return {"metric": "decode tok/s, Dimesun at production-like layer sizes (bf16), beside a like-sized GDN / attention / MoE hybrid",
            "value": first["decode_tok_s"], "unit": "tok/s", "n_gpus": 1, "ms_per_step": first["decode_ms_per_step"],
            "config": {"layers": layers, **SIZES, "head_dim": 128, "l2": "kernel inputs rotate over sets larger than L2; weights exceed L2"},
            "models": models, "kernels": rows, "gpu_launches": int(cu.LAUNCHES - l0), "data": "synthetic (seeded token ids, random-init weights)",
            "dtype": "bf16"}
