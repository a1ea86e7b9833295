"""Configurations and checks of the Begupel family that the CPU and the GPU tests share: a checkpoint is written to disk, loaded through
the registry and driven through the runner in all kinds of portions and batches, and every logit row is compared with the plain
statement in ``begupel_oracle``."""
import functools
import math

import torch

import begupel_oracle as oracle
from dimesun_cases import make_runner, portions, prompt, row_errors, save_checkpoint, error  # noqa: F401  (shared helpers)

TOL = {"float32": 8e-5, "bfloat16": 4e-2}


# ---- configurations ------------------------------------------------------------------------------------------


def left(heads, kv, dim, vdim, window, dims, base=10000.0, factor=1.0, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "mask": {"size": window},
            "rot": {"base": base, "dims": dims, "scaling": {"factor": factor}}}


def right(heads, kv, dim, vdim, conv=4):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(l, r, ls=0.7, rs=1.1):
    return "parallel", {"left": l, "right": r, "left_scale": ls, "right_scale": rs}


def lightning(heads, dim, vdim, decay=None):
    return "lightning", {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1 - 2.0 ** -(1 + 2 * h) for h in range(heads)]}


def small_config(layers, width=64, vocab=96, groups=2, eps=1e-5, taps=4, cap=20.0, bigram=(61, 13, 29)):
    """A ``config.json`` dictionary.  ``layers``: ``((type, mixer), ff or None)`` pairs."""
    return {"architecture": "Begupel", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "canon": {"taps": taps},
            "logit_softcap": cap, "embedding": {"bigram": {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}},
            "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": f} if f else None} for (t, m), f in layers]}


def _cfg_mixed():
    """Uneven sizes everywhere: shared key heads, padded heads, value sizes unlike key sizes, partial rotation, both kinds with and without
    a feed-forward, norm parts that no vector fits."""
    return small_config([(parallel(left(6, 2, 40, 56, 37, 24, base=500.0, factor=2.5), right(4, 2, 40, 24, conv=3)), 72),
                         (lightning(3, 24, 40), None), (lightning(2, 72, 136), 40),
                         (parallel(left(3, 3, 24, 16, 70, 24), right(2, 1, 24, 72, conv=5), 1.3, 0.4), None)],
                        width=72, vocab=101, groups=12, taps=3, cap=6.0)


def _cfg_wide():
    """Heads of production size, a window of one page, parts of whole warps."""
    return small_config([(lightning(2, 128, 128, [0.97, 0.9999]), 96),
                         (parallel(left(8, 2, 128, 128, 64, 128, base=1e6, factor=4.0), right(2, 2, 128, 128)), None),
                         (parallel(left(4, 4, 128, 96, 130, 64), right(4, 2, 64, 128, conv=2)), 64)], width=256, vocab=80, groups=2, taps=4)


def _cfg_ones():
    """Every size that may be one: window, taps, groups, heads, buckets' multipliers; decays of 0 and 1; large values, wide heads."""
    return small_config([(parallel(left(1, 1, 16, 200, 1, 2), right(1, 1, 16, 16, conv=1), 1.0, 1.0), 24), (lightning(3, 16, 16, [0.0, 1.0, 0.5]), None),
                         (parallel(left(2, 1, 72, 8, 20, 72, base=100.0), right(3, 1, 136, 200, conv=8), 0.5, 2.0), None)],
                        width=64, vocab=64, groups=1, eps=1e-3, taps=1, cap=5.0, bigram=(1, 1, 1))


def _cfg_long():
    """Windows that lie far inside a prompt, long convolutions in front of the mixers, a large bigram table."""
    return small_config([(lightning(2, 64, 64, [0.995, 0.8]), None), (parallel(left(4, 2, 64, 64, 100, 32), right(2, 2, 64, 64)), 64),
                         (lightning(1, 256, 64, [0.99]), None)], width=40, vocab=72, groups=4, taps=8, cap=30.0, bigram=(4099, 1000003, 8191))


CONFIGS = {"mixed": _cfg_mixed, "wide": _cfg_wide, "ones": _cfg_ones, "long": _cfg_long}


def random_weights(cfg, seed=0):
    """bfloat16 tensors of every name the design has; scaled so that activations stay near one."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s / math.sqrt(i))).bfloat16()

    def vec(n, s, off=0.0):
        return (torch.randn(n, generator=g) * s + off).bfloat16()
    d = cfg["width"]
    w = {"embed": mat(cfg["vocab"], d, d ** 0.5), "bigram": mat(cfg["embedding"]["bigram"]["buckets"] + 1, d, 0.7 * d ** 0.5),
         "head": mat(cfg["vocab"], d, 2.0), "final.norm": vec(d, 0.2, 1.0)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix"
        w[f"l{i}.norm1"] = vec(d, 0.2, 0.7)
        w[f"l{i}.canon1"] = (torch.randn(d, cfg["canon"]["taps"], generator=g) * 0.4).bfloat16()
        if l["type"] == "lightning":
            n = m["heads"]
            w[p + ".q"], w[p + ".k"], w[p + ".v"], w[p + ".g"] = mat(n * m["dim"], d), mat(n * m["dim"], d), mat(n * m["vdim"], d, 1.5), mat(n * m["vdim"], d)
            w[p + ".norm"], w[p + ".o"] = vec(n * m["vdim"], 0.2, 1.0), mat(d, n * m["vdim"], 1.5)
        else:
            a, b = m["left"], m["right"]
            p = f"l{i}.mix.left"
            w[p + ".q"], w[p + ".k"], w[p + ".v"] = mat(a["heads"] * a["dim"], d), mat(a["kv_heads"] * a["dim"], d), mat(a["kv_heads"] * a["vdim"], d, 1.5)
            w[p + ".q.norm"], w[p + ".k.norm"] = vec(a["heads"] * a["dim"], 0.2, 1.4), vec(a["kv_heads"] * a["dim"], 0.2, 1.4)
            w[p + ".o"] = mat(d, a["heads"] * a["vdim"], 1.5)
            p, n = f"l{i}.mix.right", b["heads"]
            w[p + ".q"], w[p + ".k"], w[p + ".v"] = mat(b["kv_heads"] * b["dim"], d), mat(b["kv_heads"] * b["dim"], d), mat(n * b["vdim"], d, 1.5)
            for c in "qkv":
                w[f"{p}.{c}.conv"] = (torch.randn(w[f"{p}.{c}"].shape[0], b["conv"], generator=g) * 0.6).bfloat16()
            w[p + ".b"], w[p + ".a"], w[p + ".g"] = mat(n, d, 1.5), mat(n, d, 1.5), mat(n * b["vdim"], d)
            w[p + ".A_log"], w[p + ".dt_bias"], w[p + ".norm"] = vec(n, 0.5, 0.3), vec(n, 1.5, -4.0), vec(b["vdim"], 0.2, 1.0)
            w[p + ".o"] = mat(d, n * b["vdim"], 1.5)
        if l.get("mlp"):
            f = l["mlp"]["ff"]
            w[f"l{i}.norm2"] = vec(d, 0.2, 0.7)
            for n, o, k in (("gate", f, d), ("up", f, d), ("down", d, f)):
                w[f"l{i}.mlp.{n}"], w[f"l{i}.mlp.{n}.b"] = mat(o, k, 1.5), vec(o, 0.4)
    return w


@functools.lru_cache(maxsize=None)
def weights(name: str, sharp: float = 1.0):
    """``sharp`` multiplies the score scale of the attention layers: one score per row stands out, so a key that is wrongly seen or
    wrongly hidden moves the logits."""
    cfg = CONFIGS[name]()
    for l in cfg["layers"]:
        if l["type"] == "parallel":
            l["mixer"]["left"]["scale"] *= sharp
    return cfg, random_weights(cfg, seed=sorted(CONFIGS).index(name) + 1)


@functools.lru_cache(maxsize=None)
def expected(name: str, sharp: float, n: int, seed: int):
    cfg, w = weights(name, sharp)
    return oracle.forward(cfg, w, list(prompt(cfg["vocab"], n, seed)))


def replay(runner, name, sharp, requests, steps):
    """``requests``: id → (length, seed).  ``steps``: lists of (id, count).  Returns the worst row error."""
    cfg, _ = weights(name, sharp)
    errs, at, seat_of, free = [], {}, {}, list(range(runner.kv.max_seats - 1, -1, -1))
    for step in steps:
        seats, toks, want = [], [], []
        for rid, count in step:
            n, seed = requests[rid]
            lo = at.get(rid, 0)
            if lo == 0:
                seat_of[rid] = free.pop()
            seats.append(seat_of[rid])
            toks.append(list(prompt(cfg["vocab"], n, seed)[lo:lo + count]))
            want.append(expected(name, sharp, n, seed)[lo:lo + count])
            at[rid] = lo + count
        errs.append(row_errors(runner.step(seats, toks, logits_all=True), torch.cat(want)))
        for rid, _ in step:
            if at[rid] == requests[rid][0]:
                runner.kv.free(seat_of[rid])
                free.append(seat_of.pop(rid))
    assert not seat_of, "a request was left unfinished"
    errs = torch.cat(errs)
    assert not torch.isnan(errs).any()
    return float(errs.max())


# ---- mechanisms alone, on any device -------------------------------------------------------------------------


def _pad(x, n):
    return torch.nn.functional.pad(x, (0, n - x.shape[-1]))


def _worst_row(d, w):
    """Largest root mean square of a row's difference over the scale of the values."""
    return float(d.pow(2).mean(-1).sqrt().max() / w.std())


def _steps(lens, past):
    """``(lo, hi)`` per sequence of the steps that bring every sequence to ``lens``: at once, or cut at ``past``."""
    zero = [0] * len(lens)
    return [(zero, lens)] if past is None else [(zero, past), (past, lens)]


def _rows(starts, lo, hi):
    return torch.cat([torch.arange(s + a, s + b) for s, a, b in zip(starts, lo, hi)])


def _meta(lo, hi, slots, device, table=None):
    from tensorrt_edge_llm_b200.ops.meta import build_step_meta
    live = [i for i in range(len(lo)) if hi[i] > lo[i]]
    assert len(live) == len(lo), "every sequence of a step brings rows"
    return build_step_meta([b - a for a, b in zip(lo, hi)], lo, torch.zeros(len(lo), 1, dtype=torch.int32) if table is None else table, 64,
                           slot_ids=slots, device=device)


def stream_case(device, dtype, width, groups, taps, lens, past=None, ids=False, buckets=37, mul=(1000003, 77), behind=0):
    """:func:`ops.stream_post` with a convolution: worst errors of the stream and of the convolved rows.  State rows hold leftovers.
    ``behind``: that many partial sums of squares per row, by whose root mean square (over 100 features) the update is divided."""
    from tensorrt_edge_llm_b200 import ops
    g, t, eps = torch.Generator().manual_seed(3), sum(lens), 1e-4
    starts = [sum(lens[:i]) for i in range(len(lens))]
    x, d = torch.randn(t, width, generator=g), (torch.randn(t, width, generator=g) * 3).to(dtype)
    w, conv = torch.randn(width, generator=g), torch.randn(taps, width, generator=g) * 0.5
    table, big = torch.randn(50, width, generator=g).to(dtype), torch.randn(buckets + 1, width, generator=g).to(dtype)
    toks, sums = torch.randint(0, 50, (t,), generator=g), torch.rand(t, max(behind, 1), generator=g) * 50
    f, want_x, want_h = lambda v: v.double(), [], []
    for s, n in zip(starts, lens):
        if ids:
            y = [int(v) for v in toks[s:s + n]]
            y = f(table)[y] + f(big)[oracle.bigram_rows(y, buckets, *mul)]
        else:
            y = f(d[s:s + n])
            if behind:
                y = y / torch.sqrt(f(sums[s:s + n]).sum(-1, keepdim=True) / 100 + eps)
            y = f(x[s:s + n]) + oracle.group_norm(y, f(w), groups, eps)
        want_x.append(y)
        want_h.append(y + oracle.causal_conv(y, f(conv).t()))
    dev = lambda v: v.to(device)
    hist = torch.full((6, taps - 1, width), 9.0, device=device)
    last = torch.full((6, 1), 7, dtype=torch.int32, device=device)
    slots = [4, 1, 3, 0][:len(lens)]
    got_x, got_h = torch.zeros(t, width), torch.zeros(t, width)
    for lo, hi in _steps(lens, past):
        idx = _rows(starts, lo, hi)
        kw = dict(conv=dev(conv), history=hist if taps > 1 else None)
        if ids:
            a, b = ops.stream_post(None, None, None, groups, eps, _meta(lo, hi, slots, device), dtype, ids=dev(toks[idx].int()), table=dev(table),
                                   bigram=ops.Bigram(dev(big), last, buckets, *mul), **kw)
        else:
            a, b = ops.stream_post(dev(x[idx]), dev(d[idx]), dev(w), groups, eps, _meta(lo, hi, slots, device), dtype,
                                   sums=(dev(sums[idx]), 100) if behind else None, **kw)
        got_x[idx], got_h[idx] = a.float().cpu(), b.float().cpu()
    want_x, want_h = torch.cat(want_x), torch.cat(want_h)
    return _worst_row(got_x - want_x, want_x), _worst_row(got_h - want_h, want_h)


def attention_case(device, dtype, hq, hkv, d, dv, window, dims, lens, past, factor=1.0, needle=None, mult=0.7):
    """:func:`ops.turned_kv_write` + :func:`ops.paged_attention` over caches that hold ``past`` tokens, rows and outputs inside wider
    buffers.  ``needle``: a position whose key matches every query far above all others (on a feature that does not rotate): rows
    whose window holds it return its value, turned by the distance."""
    from tensorrt_edge_llm_b200 import ops
    from tensorrt_edge_llm_b200.config import AttentionConfig
    base, eps = 1000.0, 1e-4
    sp = AttentionConfig(hq, hkv, d, dv, dims, base, 2.0 * d ** -0.5, window=window, row_norm=True, interleaved=True, rope_factor=factor, rotated_values=True)
    g, total = torch.Generator().manual_seed(5), [a + b for a, b in zip(lens, past)]
    n_all, c = sum(total), {"rot": {"dims": dims, "base": base, "scaling": {"factor": factor}}, "scale": sp.scale, "mask": {"size": window}}
    q, k, v = torch.randn(n_all, hq, d, generator=g), torch.randn(n_all, hkv, d, generator=g), torch.randn(n_all, hkv, dv, generator=g)
    qw, kw = torch.randn(hq * d, generator=g) * 0.2 + 1, torch.randn(hkv * d, generator=g) * 0.2 + 1
    starts = [sum(total[:i]) for i in range(len(lens))]
    if needle is not None:
        assert dims < d
        q[:, :, -1], k[:, :, -1] = 8.0 * d ** 0.5, 0.0
        qw.view(hq, d)[:, -1], kw.view(hkv, d)[:, -1] = 1.5, 1.5
        at = [s + needle for s, n in zip(starts, total) if needle < n]
        k[at] = 0.0
        k[at, :, -1] = 1.0                                   # small: only its direction counts
    q, k, v = (x.to(dtype) for x in (q, k, v))
    f, want = lambda x: x.double(), []
    for s, n, p0 in zip(starts, total, past):
        rows = slice(s, s + n)
        qq = oracle.rms_norm(f(q[rows]).reshape(n, -1), eps, f(qw)).reshape(n, hq, d)
        kk = oracle.rms_norm(f(k[rows]).reshape(n, -1), eps, f(kw)).reshape(n, hkv, d)
        want.append(oracle.attention_heads(qq, kk, f(v[rows]), c)[p0:] * mult)
    pad, per = sp.pad, (max(total) + 63) // 64
    wide = torch.randn(n_all, (hq + 2 * hkv) * pad + 64, generator=g).to(dtype)                    # the rows lie in a wider product
    wide[:, :-64] = torch.cat([_pad(x, pad).reshape(n_all, -1) for x in (q, k, v)], -1)
    table = torch.randperm(per * len(lens) + 2, generator=g)[:per * len(lens)].reshape(len(lens), per).to(torch.int32)
    cache = torch.randn(per * len(lens) + 2, 2, hkv, 64, pad, generator=g).to(dtype).to(device)     # leftovers of earlier requests
    dev = lambda x: x.to(device)
    scaling = None if factor == 1.0 else {"rope_type": "linear", "factor": factor}
    keys = ops.rope_cos_sin(max(total), dims, base, scaling, device=device, pairs=pad // 2)
    values = ops.rope_cos_sin(max(total), dv, base, None, device=device, pairs=pad // 2)
    norms = [dev(_pad(w.reshape(h, d), pad).reshape(-1)) for w, h in ((qw, hq), (kw, hkv))]
    for lo, hi in (([0] * len(lens), past), (past, total)):
        if not any(hi):
            continue
        seqs = [i for i in range(len(lens)) if hi[i] > lo[i]]
        meta = _meta([lo[i] for i in seqs], [hi[i] for i in seqs], None, device, table[seqs])
        idx = _rows([starts[i] for i in seqs], [lo[i] for i in seqs], [hi[i] for i in seqs])
        qn = ops.turned_kv_write(dev(wide[idx])[:, :-64], cache, meta, keys, values, *norms, sp, eps)
    buf = torch.full((sum(lens), hq * pad + 32), 5.0, dtype=dtype, device=device)
    ops.paged_attention(qn, cache, meta, sp.scale, window, fp32_weights=True, back=(values, mult), out=buf[:, :hq * pad])
    assert float(buf[:, hq * pad:].float().min()) == 5.0
    got = buf[:, :hq * pad].float().cpu().view(-1, hq, pad)
    assert pad == dv or float(got[:, :, dv:].abs().max()) == 0.0
    w = torch.cat(want)
    if needle is not None:                                   # the case is sharp: rows that see the needle return (almost) its value alone
        pos = torch.cat([torch.arange(p0, n) for n, p0 in zip(total, past)])
        seen = (pos >= needle) & (pos - needle < window)
        one = torch.cat([f(v[[s + needle] * m]) if needle < s_n else torch.zeros(m, hkv, dv, dtype=torch.float64)
                         for s, s_n, m in zip(starts, total, lens)])
        size = one.pow(2).sum((1, 2)).sqrt() * mult * (hq / hkv) ** 0.5
        near = (w.pow(2).sum((1, 2)).sqrt() / size.clamp_min(1e-9) - 1).abs() < 0.05
        assert bool(near[seen].all())
    return _worst_row(got[:, :, :dv].double() - w, w)


def delta_case(device, dtype, heads, kv, dk, dv, conv, lens, past=None, kernel=None, keep=-1, mult=1.3):
    """Rows for :func:`ops.channel_delta` with one decay per head and a silu gate, at padded sizes and inside wider products, against the
    recurrence of the oracle; ``past`` cuts every sequence once.  ``keep``: a token with step size one, decays of one and no other
    writes: its value must stay in the state."""
    from tensorrt_edge_llm_b200 import ops
    from tensorrt_edge_llm_b200.config import ChannelDeltaConfig
    sp = ChannelDeltaConfig(heads, kv, dk, dv, conv, 0, 0, head_decay=True, silu_gate=True)
    kp, vp, t, eps = sp.k_pad, sp.v_pad, sum(lens), 1e-5
    g = torch.Generator().manual_seed(7)
    q, k, v = torch.randn(t, kv, dk, generator=g), torch.randn(t, kv, dk, generator=g), torch.randn(t, heads, dv, generator=g)
    z, gate, beta = torch.randn(t, heads, generator=g) * 1.5, torch.randn(t, heads, dv, generator=g), torch.randn(t, heads, generator=g)
    if keep >= 0:
        z[:], beta[:] = -30.0, -30.0
        beta[keep::max(lens)] = 30.0
    taps = [(torch.randn(n * d, conv, generator=g) * 0.6).to(dtype) for n, d in ((kv, dk), (kv, dk), (heads, dv))]
    a_log, bias, nw = torch.randn(heads, generator=g) * 0.5, torch.randn(heads, generator=g) - 3.0, torch.randn(dv, generator=g) * 0.2 + 1
    q, k, v, gate = (x.to(dtype) for x in (q, k, v, gate))
    cols = [_pad(q, kp).reshape(t, -1), _pad(k, kp).reshape(t, -1), _pad(v, vp).reshape(t, -1), _pad(gate, vp).reshape(t, -1)]
    wide = torch.cat([torch.randn(t, 64, generator=g).to(dtype)] + cols, -1)
    small = torch.cat([beta, z], -1)
    conv_w = torch.cat([torch.nn.functional.pad(w.reshape(n, d, conv), (0, 0, 0, p - d)).reshape(n * p, conv)
                        for w, n, d, p in zip(taps, (kv, kv, heads), (dk, dk, dv), (kp, kp, vp))])
    want, f, starts = [], lambda x: x.double(), [sum(lens[:i]) for i in range(len(lens))]
    for s, n in zip(starts, lens):
        rows = slice(s, s + n)
        y = [oracle.silu(oracle.causal_conv(f(x[rows]).reshape(n, -1), f(w))).to(dtype).double().reshape(n, -1, d)
             for x, w, d in zip((q, k, v), taps, (dk, dk, dv))]
        rep = heads // kv
        o = oracle.delta_recurrence((oracle.unit(y[0]) * dk ** -0.5).repeat_interleave(rep, 1), oracle.unit(y[1]).repeat_interleave(rep, 1), y[2],
                                    oracle.head_decay(f(z[rows]), f(a_log), f(bias)), torch.sigmoid(f(beta[rows])))
        want.append(oracle.rms_norm(o, eps, f(nw)) * oracle.silu(f(gate[rows])) * mult)
    conv_state = torch.full((6, sp.conv_dim, conv - 1), 9.0, dtype=dtype, device=device)          # rows hold leftovers of earlier requests
    state = torch.full((6, heads, kp, vp), 9.0, device=device)
    slots = [4, 1, 3, 0][:len(lens)]
    fn = ops.channel_delta if kernel is None else functools.partial(ops.cuda_ops().channel_delta, kernel=kernel)
    dev = lambda x: x.to(device)
    got = torch.zeros(t, heads, vp)
    for lo, hi in _steps(lens, past):
        idx = _rows(starts, lo, hi)
        rows, sm = dev(wide[idx]), dev(small[idx])
        buf = torch.full((len(idx), heads * vp + 64), 5.0, dtype=dtype, device=device)
        c = 64 + sp.conv_dim
        fn(rows[:, 64:c], sm[:, heads:], rows[:, c:], sm[:, :heads], dev(conv_w), dev(a_log), dev(bias), dev(_pad(nw, vp)), conv_state, state,
           _meta(lo, hi, slots, device), sp, eps, out=buf[:, 64:], mult=mult)
        assert float(buf[:, :64].float().min()) == 5.0
        got[idx] = buf[:, 64:].float().cpu().view(-1, heads, vp)
    assert vp == dv or float(got[:, :, dv:].abs().max()) == 0.0
    w = torch.cat(want)
    if keep >= 0:                                            # the kept value is what every later row of its sequence reads out
        assert float(w[keep + 1:lens[0]].abs().max()) > 1e-3
    return float((got[:, :, :dv].double() - w).pow(2).mean().sqrt() / w.std())


def lightning_case(device, dtype, heads, dk, dv, lens, past=None, decay=None, kernel=None, loud=None, **force):
    """:func:`ops.lightning` at padded sizes against the memory of the oracle: worst row error of the normed outputs, and the error of the
    states.  ``loud``: a row whose key and value are large, so that it has to be carried (decayed) through every later row."""
    from tensorrt_edge_llm_b200 import ops
    from tensorrt_edge_llm_b200.config import LightningConfig
    decay = decay or [1 - 2.0 ** -(2 + 3 * h) for h in range(heads)]
    sp = LightningConfig(heads, dk, dv, decay)
    kp, vp, t, eps = sp.k_pad, sp.v_pad, sum(lens), 1e-5
    g = torch.Generator().manual_seed(9)
    q, k = torch.randn(t, heads, dk, generator=g), torch.randn(t, heads, dk, generator=g)
    v, gate, nw = torch.randn(t, heads, dv, generator=g), torch.randn(t, heads, dv, generator=g), torch.randn(heads, dv, generator=g) * 0.2 + 1
    starts = [sum(lens[:i]) for i in range(len(lens))]
    if loud is not None:
        at = [s + loud for s, n in zip(starts, lens) if loud < n]
        k[at], v[at] = 6.0, 8.0
    q, k, v, gate = (x.to(dtype) for x in (q, k, v, gate))
    f, want, states = lambda x: x.double(), [], []
    act = lambda x: oracle.silu(f(x)).to(dtype).double()
    dd = torch.tensor(decay, dtype=torch.float64)
    for s, n in zip(starts, lens):
        rows = slice(s, s + n)
        o = oracle.decayed_memory(act(q[rows]), act(k[rows]), act(v[rows]), dd).reshape(n, -1)
        want.append(oracle.rms_norm(o, eps, f(nw).reshape(-1)) * torch.sigmoid(f(gate[rows]).reshape(n, -1)))
        age = dd[None] ** torch.arange(n - 1, -1, -1, dtype=torch.float64)[:, None]
        states.append(torch.einsum("th,thd,thv->hdv", age, act(k[rows]), act(v[rows])))
    packed = torch.cat([_pad(q, kp).reshape(t, -1), _pad(k, kp).reshape(t, -1), _pad(v, vp).reshape(t, -1), _pad(gate, vp).reshape(t, -1)], -1)
    powers = (dd[:, None] ** torch.arange(257, dtype=torch.float64)).float()
    state = torch.full((6, heads, kp, vp), 9.0, device=device)
    slots = [4, 1, 3, 0, 5, 2][:len(lens)]
    if kernel is not None:
        force["kernel"] = kernel
    fn = functools.partial(ops.cuda_ops().lightning, **force) if force else ops.lightning
    dev, got = (lambda x: x.to(device)), torch.zeros(t, heads, vp)
    for lo, hi in _steps(lens, past):
        idx = _rows(starts, lo, hi)
        u, sums = fn(dev(packed[idx]), dev(_pad(nw, vp).reshape(-1)), dev(powers), state, _meta(lo, hi, slots, device))
        rms = torch.sqrt(sums.double().cpu().sum(-1) / (heads * dv) + eps)
        got[idx] = (u.double().cpu() / rms[:, None]).float().view(-1, heads, vp)
    assert vp == dv or float(got[:, :, dv:].abs().max()) == 0.0
    w, st = torch.cat(want), torch.stack(states)
    err = torch.stack([(state[s].cpu().double()[:, :dk, :dv] - x).pow(2).mean((-1, -2)).sqrt() / x.pow(2).mean((-1, -2)).sqrt() for s, x in zip(slots, st)])
    return _worst_row(got[:, :, :dv].reshape(t, -1).double() - w, w), float(err.max())
