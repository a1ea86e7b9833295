"""Configurations and checks of the Ditenex family that the CPU and the GPU tests share: a checkpoint is written to disk, loaded through
the registry and driven through the runner in all kinds of portions and batches, and every logit row is compared with the plain
statement in ``ditenex_oracle``."""
import functools
import math

import torch

import ditenex_oracle as oracle
from dimesun_cases import error, make_runner, portions, prompt, row_errors, save_checkpoint  # noqa: F401  (shared helpers)

TOL = {"float32": 8e-5, "bfloat16": 2e-2}


# ---- configurations ------------------------------------------------------------------------------------------


def attn(heads, kv, dim, vdim, window, v_mix=True, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "mask": {"size": window}, "v_mix": v_mix}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, count, keep, scale=1.5, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}
    return {**out, "shared": {"ff": shared}} if shared else out


def small_config(layers, width=64, vocab=96, eps=1e-5, mult=0.4, positions=400):
    """A ``config.json`` dictionary.  ``layers``: ``(mixer, feed-forward or None)`` pairs."""
    return {"architecture": "Ditenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "max_positions": positions,
            "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}


def _cfg_mixed():
    """Uneven sizes everywhere: padded heads, value sizes unlike key sizes, three query heads per KV head; the first layer does not mix
    values and one in between neither; layers that mix values pad their heads differently; a layer without a feed-forward, experts with and without a shared one."""
    return small_config([(attn(6, 2, 40, 56, 37, v_mix=False), dense(72)), (attn(6, 3, 40, 24, 20), moe(9, 3, 40, 3, 2, 1.7, 48)),
                         (attn(3, 3, 24, 24, 70), None), (attn(2, 1, 72, 16, 33, v_mix=False), moe(6, 2, 24, 2, 1, 2.5)),
                         (attn(12, 3, 72, 24, 90), dense(40))], width=72, vocab=101)


def _cfg_wide():
    """Heads of production size, a window of one page, sixteen heads on four KV heads."""
    return small_config([(attn(16, 4, 128, 128, 64), dense(96)), (attn(8, 4, 64, 128, 130), moe(16, 4, 64, 4, 2, 2.0, 64)),
                         (attn(4, 4, 128, 128, 200), dense(64))], width=256, vocab=80, mult=0.3)


def _cfg_ones():
    """Every size that may be one: window, heads, experts, groups, multipliers; heads wider than the tensor-core kernels take."""
    return small_config([(attn(1, 1, 16, 200, 1, scale=1.0), dense(24)), (attn(3, 1, 130, 200, 17), moe(1, 1, 16, 1, 1, 1.0, 8)),
                         (attn(2, 1, 8, 200, 5), moe(4, 1, 8, 4, 1, 1.0))], width=64, vocab=64, eps=1e-3, mult=1.0)


def _cfg_long():
    """Windows that lie far inside a prompt, one key head for all, as many key heads as query heads, experts of which all are used."""
    return small_config([(attn(8, 1, 80, 64, 100), moe(4, 4, 24, 2, 2, 0.7, 24)), (attn(4, 2, 64, 40, 300, v_mix=False), dense(64)),
                         (attn(5, 1, 64, 64, 65), None), (attn(10, 10, 48, 32, 50, v_mix=False), dense(32))], width=40, vocab=72, mult=0.6)


CONFIGS = {"mixed": _cfg_mixed, "wide": _cfg_wide, "ones": _cfg_ones, "long": _cfg_long}


def random_weights(cfg, seed=0):
    """bfloat16 tensors of every name the design has; scaled so that activations stay near one.  Corrections are negative, so choice scores
    are, and router logits spread so that few choices are close."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s / math.sqrt(i))).bfloat16()

    def vec(n, s, off=0.0):
        return (torch.randn(n, generator=g) * s + off).bfloat16()
    d = cfg["width"]
    w = {"embed": mat(cfg["vocab"], d, d ** 0.5), "pos": mat(cfg["max_positions"], d, 0.7 * d ** 0.5), "final.norm": vec(d, 0.2, 0.3)}
    for i, l in enumerate(cfg["layers"]):
        m, p, n = l["mixer"], f"l{i}.mix", l["mixer"]["heads"]
        for name in ("norm1", "norm1b"):
            w[f"l{i}.{name}"] = vec(d, 0.2, 1.0)
        w[f"l{i}.shift"] = torch.rand(d, generator=g).bfloat16()
        for c, rows, s in (("q", n * m["dim"], 1.2), ("k", m["kv_heads"] * m["dim"], 1.2), ("v", m["kv_heads"] * m["vdim"], 1.5)):
            w[f"{p}.{c}"], w[f"{p}.{c}.b"] = mat(rows, d, s), vec(rows, 0.5)
        w[p + ".g"], w[p + ".o"] = mat(n * m["vdim"], d, 1.5), mat(d, n * m["vdim"], 1.5)
        w[p + ".talk"] = (torch.eye(n) + torch.randn(n, n, generator=g) * 0.4).bfloat16()
        w[p + ".vmix"] = (torch.rand((), generator=g) * 0.5 + 0.3).bfloat16()
        f, q = l.get("mlp"), f"l{i}.mlp"
        if not f:
            continue
        for name in ("norm2", "norm2b"):
            w[f"l{i}.{name}"] = vec(d, 0.2, 1.0)
        if f["kind"] == "dense":
            w[q + ".up"], w[q + ".down"], w[q + ".act"] = mat(f["ff"], d, 1.5), mat(d, f["ff"], 1.5), torch.tensor([0.8, -0.6]).bfloat16()
            continue
        units = [(f"{q}.e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + ([(q + ".shared", f["shared"]["ff"])] if f.get("shared") else [])
        for name, size in units:
            w[name + ".gate"], w[name + ".up"], w[name + ".down"] = mat(size, d, 1.5), mat(size, d, 1.5), mat(d, size, 1.5)
        w[q + ".router"], w[q + ".correction"] = mat(f["router"]["experts"], d, 3.0), vec(f["router"]["experts"], 0.2, -1.3)
    return w


@functools.lru_cache(maxsize=None)
def weights(name: str, sharp: float = 1.0):
    """``sharp`` multiplies the score scale of the attention layers: one score per row stands out, so a key that is wrongly seen or
    wrongly hidden moves the logits."""
    cfg = CONFIGS[name]()
    for l in cfg["layers"]:
        l["mixer"]["scale"] *= sharp
    return cfg, random_weights(cfg, seed=sorted(CONFIGS).index(name) + 1)


@functools.lru_cache(maxsize=None)
def expected(name: str, sharp: float, n: int, seed: int):
    cfg, w = weights(name, sharp)
    return oracle.forward(cfg, w, list(prompt(cfg["vocab"], n, seed)))


def replay(runner, name, sharp, requests, steps):
    """``requests``: id → (length, seed).  ``steps``: lists of (id, count).  The row error that has to stay below the tolerance: the worst one in
    32 bits, the ninth decile in 16 bits (rounding flips close choices of experts)."""
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
        at = {r: c for r, c in at.items() if c < requests[r][0]}
    assert not seat_of, "a request was left unfinished"
    errs = torch.cat(errs)
    assert not torch.isnan(errs).any()
    return float(errs.max() if runner.model.cfg.dtype == "float32" else errs.quantile(0.9))


# ---- mechanisms alone, on any device -------------------------------------------------------------------------


def _pad(x, n):
    return torch.nn.functional.pad(x, (0, n - x.shape[-1]))


def _worst_row(d, w):
    """Largest root mean square of a row's difference over the scale of the values."""
    return float(d.pow(2).mean(-1).sqrt().max() / w.std())


def _rows(starts, lo, hi):
    return torch.cat([torch.arange(s + a, s + b) for s, a, b in zip(starts, lo, hi)])


def _meta(lo, hi, slots, device, table=None):
    from tensorrt_edge_llm_b200.ops.meta import build_step_meta
    return build_step_meta([b - a for a, b in zip(lo, hi)], lo, torch.zeros(len(lo), 1, dtype=torch.int32) if table is None else table, 64,
                           slot_ids=slots, device=device)


def sandwich_case(device, dtype, width, lens, past=None, ids=False, shift=True, top=0, dense=True, mult=0.7, eps=1e-4):
    """:func:`ops.stream_sandwich`: worst errors of the stream and of the (shifted) normed rows.  State rows hold leftovers.  ``top``: that many
    expert rows per token join the update, from a table in another order."""
    from tensorrt_edge_llm_b200 import ops
    g, t = torch.Generator().manual_seed(3), sum(lens)
    rnd = lambda *s: torch.randn(*s, generator=g)
    starts, f = [sum(lens[:i]) for i in range(len(lens))], lambda v: v.double()
    x, d, post, norm, amount = rnd(t, width), (rnd(t, width) * 3).to(dtype), rnd(width), rnd(width), torch.rand(width, generator=g) * 1.5
    table, positions = rnd(50, width).to(dtype), rnd(max(lens) + 1, width).to(dtype)
    toks = torch.randint(0, 50, (t,), generator=g)
    order, weight = torch.randperm(t * max(top, 1) + 7, generator=g)[:t * max(top, 1)].reshape(t, -1), torch.rand(t, max(top, 1), generator=g) + 0.2
    expert = (rnd(t * max(top, 1) + 7, width) * 2).to(dtype)
    want_x, want_h = [], []
    for s, n in zip(starts, lens):
        rows = slice(s, s + n)
        if ids:
            y = f(table)[toks[rows]] + f(positions)[:n]
        else:
            u = (f(d[rows]) if dense else 0.0) + ((f(expert)[order[rows]] * f(weight[rows])[:, :, None]).sum(1) if top else 0.0)
            y = f(x[rows]) + mult * oracle.rms_norm(u, eps, f(post))
        want_x.append(y)
        h = oracle.rms_norm(y, eps, f(norm))
        want_h.append(oracle.token_shift(h, f(amount)) if shift else h)
    dev, state = (lambda v: v.to(device)), torch.full((6, 1, width), 9.0, device=device)
    slots = [4, 1, 3, 0][:len(lens)]
    got_x, got_h = torch.zeros(t, width), torch.zeros(t, width)
    zero = [0] * len(lens)
    for lo, hi in [(zero, lens)] if past is None else [(zero, past), (past, lens)]:
        idx = _rows(starts, lo, hi)
        kw = dict(norm=dev(norm), shift=dev(amount) if shift else None, state=state if shift else None)
        if ids:
            kw.update(ids=dev(toks[idx].int()), table=dev(table), positions=dev(positions))
        else:
            routed = None
            if top and device == "cpu":
                routed = (expert[order[idx]].float() * weight[idx][:, :, None]).sum(1)
            elif top:
                from types import SimpleNamespace

                from tensorrt_edge_llm_b200.models.qwen3_moe import RoutedRows
                routed = RoutedRows(dev(expert), SimpleNamespace(dst_row=dev(order[idx].int().reshape(-1).contiguous())), dev(weight[idx]))
            kw.update(delta=dev(d[idx]) if dense else None, routed=routed, post=dev(post), mult=mult)
        a, b = ops.stream_sandwich(None if ids else dev(x[idx]), eps, _meta(lo, hi, slots, device), dtype, **kw)
        got_x[idx], got_h[idx] = a.float().cpu(), b.float().cpu()
    want_x, want_h = torch.cat(want_x), torch.cat(want_h)
    return _worst_row(got_x - want_x, want_x), _worst_row(got_h - want_h, want_h)


def attention_case(device, dtype, heads, kv, d, dv, window, lens, past, needle=None, kernel=None, join=True, gate=True, loud=1.0, **force):
    """:func:`ops.mixed_kv_write` + :func:`ops.mixed_attention` over caches that hold ``past`` tokens, rows inside wider products.  ``needle``: a
    position whose key matches every query far above all others (and above the distance bias): rows whose window holds it return its
    value.  ``loud`` multiplies the scores; ``join``: values join with another layer's."""
    from tensorrt_edge_llm_b200 import ops
    from tensorrt_edge_llm_b200.config import AttentionConfig
    sp = AttentionConfig(heads, kv, d, dv, 0, scale=loud * d ** -0.5, window=window, mixed_scores=True, distance_bias=True, value_mix=join, qkv_bias=True, out_gate=gate)
    g, total = torch.Generator().manual_seed(5), [a + b for a, b in zip(lens, past)]
    n_all, pad = sum(total), sp.pad
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, k, v, first, z = rnd(n_all, heads, d), rnd(n_all, kv, d), rnd(n_all, kv, dv), rnd(n_all, kv, dv), rnd(n_all, heads, dv)
    mix, share = torch.eye(heads) + rnd(heads, heads) * 0.4, torch.tensor(0.3)
    starts = [sum(total[:i]) for i in range(len(lens))]
    if needle is not None:
        mix = mix.abs() / mix.abs().sum(1, keepdim=True)         # the needle's score survives the mixing of equal scores
        k[:, :, -1], q[:, :, -1] = 0.0, 400.0 * d ** 0.5 / loud
        at = [s + needle for s, n in zip(starts, total) if needle < n]
        k[at] = 0.0
        k[at, :, -1] = 1.0
    q, k, v, first, z = (x.to(dtype) for x in (q, k, v, first, z))
    f, want = lambda x: x.double(), []
    for s, n, p0 in zip(starts, total, past):
        rows = slice(s, s + n)
        val = oracle.mix_values(f(v[rows]), f(first[rows]), float(share)) if join else f(v[rows])
        o = oracle.attend(f(q[rows]), f(k[rows]), val, f(mix), sp.scale, window)
        if needle is not None and needle < n:                    # the case is sharp: rows that see the needle return its value
            seen = [i for i in range(n) if 0 <= i - needle < window]
            assert float((o[seen] - val[needle].repeat_interleave(heads // kv, 0)).abs().max()) < 1e-2
        want.append((o * torch.sigmoid(f(z[rows])) if gate else o)[p0:])
    per = (max(total) + 63) // 64
    cols = [_pad(x, pad).reshape(n_all, -1) for x in (q, k, v, z)]
    wide, other = torch.cat(cols, -1), torch.cat([_pad(first, pad).reshape(n_all, -1), rnd(n_all, 64).to(dtype)], -1)
    table = torch.randperm(per * len(lens) + 2, generator=g)[:per * len(lens)].reshape(len(lens), per).to(torch.int32)
    cache = rnd(per * len(lens) + 2, 2, kv, 64, pad).to(dtype).to(device)                          # leftovers of earlier requests
    dev = lambda x: x.to(device)
    slope = (mix.double() @ oracle.distance_slopes(heads)).float()
    run = ops.mixed_attention if kernel is None and not force else functools.partial(ops.cuda_ops().mixed_attention, kernel=kernel, **force)
    for lo, hi in (([0] * len(lens), past), (past, total)):
        if not any(hi):
            continue
        seqs = [i for i in range(len(lens)) if hi[i] > lo[i]]
        meta = _meta([lo[i] for i in seqs], [hi[i] for i in seqs], None, device, table[seqs])
        idx = _rows([starts[i] for i in seqs], [lo[i] for i in seqs], [hi[i] for i in seqs])
        rows = dev(wide[idx])
        qn = ops.mixed_kv_write(rows, cache, meta, dev(mix), dev(other[idx])[:, :-64] if join else None, dev(share), sp)
    got = run(qn, cache, meta, dev(slope), rows[:, (heads + 2 * kv) * pad:] if gate else None, sp).float().cpu().view(-1, heads, pad)
    assert pad == dv or float(got[:, :, dv:].abs().max()) == 0.0
    w = torch.cat(want)
    return _worst_row(got[:, :, :dv].double() - w, w)
