"""Configurations and checks of the Debonex family that the CPU and the GPU tests share: a checkpoint is written to disk, loaded through
the registry and driven through the runner in all kinds of portions and batches, and every logit row is compared with the plain
statement in ``debonex_oracle``."""
import functools

import torch

import debonex_oracle as oracle
from debonex_oracle import attn_mixer, delta_mixer, latent_mixer, small_config
from dimesun_cases import make_runner, portions, prompt, row_errors, save_checkpoint, error  # noqa: F401  (shared helpers)

TOL = {"float32": 5e-5, "bfloat16": 4e-2}


def _cfg_mixed():
    """Uneven sizes everywhere: shared q / k heads, padded heads, value heads unlike key heads, a layer without a feed-forward."""
    return small_config([("channel_delta", delta_mixer(4, 2, 40, 24, conv=3), 72), ("latent_attention", latent_mixer(3, 40, 24, 56, 72, base=500.0), 40),
                         ("attention", attn_mixer(6, 2, 48, 80, coef=0.4, every=30), None), ("channel_delta", delta_mixer(2, 2, 64, 96, conv=4), 136)],
                        width=72, vocab=101)


def _cfg_latent():
    """Latents at production sizes, more columns than one block, a rank that is no multiple of 128."""
    return small_config([("latent_attention", latent_mixer(16, 128, 64, 128, 512), 64), ("latent_attention", latent_mixer(5, 64, 32, 64, 192, base=1e5), None)],
                        width=64, vocab=80, emb=1.0, logit_scale=0.5)


def _cfg_delta():
    """Single and wide heads, long and one-tap convolutions, three value heads per q / k head."""
    return small_config([("channel_delta", delta_mixer(2, 1, 136, 200, conv=8), 48), ("channel_delta", delta_mixer(1, 1, 16, 16, conv=1), None),
                         ("channel_delta", delta_mixer(3, 1, 128, 128, conv=2), 32), ("channel_delta", delta_mixer(3, 3, 128, 128), None)],
                        width=96, vocab=64, eps=1e-3)


def _cfg_attention():
    return small_config([("attention", attn_mixer(8, 2, 128, 128, coef=0.6, every=7), 64), ("attention", attn_mixer(4, 4, 200, 32, coef=0.2, every=64), 24),
                         ("attention", attn_mixer(2, 1, 24, 64, coef=0.0, every=1), None)], width=96, vocab=72)


CONFIGS = {"mixed": _cfg_mixed, "latent": _cfg_latent, "delta": _cfg_delta, "attention": _cfg_attention}


@functools.lru_cache(maxsize=None)
def weights(name: str, sharp: float = 1.0):
    """``sharp`` multiplies the score scale of the attention layers: one score per row stands out, so a key that is wrongly seen or
    wrongly hidden moves the logits."""
    cfg = CONFIGS[name]()
    for l in cfg["layers"]:
        if "scale" in l["mixer"]:
            l["mixer"]["scale"] *= sharp
    return cfg, oracle.random_weights(cfg, seed=sorted(CONFIGS).index(name) + 1)


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


# ---- mechanisms alone, on any device --------------------------------------------------------------------------------------------


def delta_case(device, dtype, heads, kv, dk, dv, conv, lens, past=None, kernel=None, keep=-1):
    """Packed rows for :func:`ops.channel_delta` at padded sizes against the recurrence of the oracle over the same numbers; ``past`` cuts
    every sequence once.  ``keep``: a token with step size one whose key does not decay afterwards (it must stay in the state)."""
    from tensorrt_edge_llm_b200 import ops
    from tensorrt_edge_llm_b200.config import ChannelDeltaConfig
    from tensorrt_edge_llm_b200.ops.meta import build_step_meta
    sp = ChannelDeltaConfig(heads, kv, dk, dv, conv)
    kp, vp, t, eps = sp.k_pad, sp.v_pad, sum(lens), 1e-5
    g = torch.Generator().manual_seed(7)
    pad = lambda x, n: torch.nn.functional.pad(x, (0, n - x.shape[-1]))
    q, k, v = torch.randn(t, kv, dk, generator=g), torch.randn(t, kv, dk, generator=g), torch.randn(t, heads, dv, generator=g)
    z, gate, beta = torch.randn(t, heads, dk, generator=g) * 1.5, torch.randn(t, heads, dv, generator=g), torch.randn(t, heads, generator=g)
    if keep >= 0:
        z[:] = -30.0
        beta[:] = -30.0
        beta[keep::max(lens)] = 30.0
    taps = [torch.randn(n * d, conv, generator=g) * 0.6 for n, d in ((kv, dk), (kv, dk), (heads, dv))]
    a_log, bias, nw = torch.randn(heads, generator=g) * 0.5, torch.randn(heads, dk, generator=g) - 3.0, torch.randn(dv, generator=g) * 0.2 + 1
    q, k, v, gate = (x.to(dtype) for x in (q, k, v, gate))
    taps = [x.to(dtype) for x in taps]
    qkv = torch.cat([pad(q, kp).reshape(t, -1), pad(k, kp).reshape(t, -1), pad(v, vp).reshape(t, -1)], -1)
    conv_w = torch.cat([torch.nn.functional.pad(w.reshape(n, d, conv), (0, 0, 0, p - d)).reshape(n * p, conv)
                        for w, n, d, p in zip(taps, (kv, kv, heads), (dk, dk, dv), (kp, kp, vp))])
    want, r0, f = [], 0, lambda x: x.double()
    for n in lens:
        rows = slice(r0, r0 + n)
        y = [oracle.silu(oracle.short_conv(f(x[rows]).reshape(n, -1), f(w))).to(dtype).double().reshape(n, -1, d)
             for x, w, d in zip((q, k, v), taps, (dk, dk, dv))]
        dec = torch.exp(-torch.exp(f(a_log))[:, None] * torch.nn.functional.softplus(f(z[rows]) + f(bias)))
        rep = heads // kv
        o = torch.stack([oracle.delta_recurrence(oracle.unit(y[0][:, h // rep]) * dk ** -0.5, oracle.unit(y[1][:, h // rep]), y[2][:, h], dec[:, h],
                                                 torch.sigmoid(f(beta[rows, h]))) for h in range(heads)], 1)
        want.append(oracle.rms_norm(o, eps, f(nw)) * torch.sigmoid(f(gate[rows])))
        r0 += n
    conv_state = torch.full((6, sp.conv_dim, conv - 1), 9.0, dtype=dtype, device=device)          # rows hold leftovers of earlier requests
    state = torch.full((6, heads, kp, vp), 9.0, device=device)
    slots, table = [4, 1, 3, 0][:len(lens)], torch.zeros(len(lens), 1, dtype=torch.int32)
    fn = ops.channel_delta if kernel is None else functools.partial(ops.cuda_ops().channel_delta, kernel=kernel)
    dev = lambda x: x.to(device)
    starts = [sum(lens[:i]) for i in range(len(lens))]
    cuts = [[0] * len(lens), lens] if past is None else [[0] * len(lens), past, lens]
    got = torch.zeros(t, heads, vp)
    for lo, hi in zip(cuts, cuts[1:]):
        idx = torch.cat([torch.arange(s + a, s + b) for s, a, b in zip(starts, lo, hi)])
        meta = build_step_meta([b - a for a, b in zip(lo, hi)], lo, table, 64, slot_ids=slots, device=device)
        out = fn(dev(qkv[idx]), dev(pad(z, kp).reshape(t, -1)[idx]), dev(pad(gate, vp).reshape(t, -1)[idx]), dev(beta[idx]), dev(conv_w), dev(a_log),
                 dev(pad(bias, kp).reshape(-1)), dev(pad(nw, vp)), conv_state, state, meta, sp, eps)
        got[idx] = out.float().cpu().view(-1, heads, vp)
    assert vp == dv or float(got[:, :, dv:].abs().max()) == 0.0
    w = torch.cat(want)
    if keep >= 0:                                            # the kept value is what every later row of its sequence reads out
        assert float(w[keep + 1:lens[0]].abs().max()) > 1e-3
    return float((got[:, :, :dv].double() - w).pow(2).mean().sqrt() / w.std())


def latent_case(device, dtype, heads, dim, rot, dv, rank, lens, past, kernel=None, needle=None, scale=None):
    """A step of :func:`ops.latent_write` + :func:`ops.latent_attention` over caches that hold ``past`` tokens.  ``needle``: a position whose
    key matches every query far above all others: rows that see it must return its value, earlier rows must not."""
    from tensorrt_edge_llm_b200 import ops
    from tensorrt_edge_llm_b200.config import LatentConfig
    from tensorrt_edge_llm_b200.ops.meta import build_step_meta
    sp = LatentConfig(heads, dim, rot, dv, rank, 1000.0, scale or (dim + rot) ** -0.5)
    g = torch.Generator().manual_seed(11)
    eps, total = 1e-5, [a + b for a, b in zip(lens, past)]
    n_all = sum(total)
    q, kv = torch.randn(n_all, heads, dim + rot, generator=g), torch.randn(n_all, rank + rot, generator=g)
    uk, uv = torch.randn(heads, dim, rank, generator=g) * rank ** -0.5, torch.randn(heads, dv, rank, generator=g) * rank ** -0.5
    if needle is not None:
        # one latent direction carries the match: only the needle's latent has it, and every query looks for it
        kv[:, 0] = 0.0
        uk[:, :, 0] = 0.0
        uk[:, 0, 0], q[:, :, 0] = 1.0, 12.0
        q[:, :, 1:] *= 0.1
        at = [sum(total[:i]) + needle for i in range(len(lens)) if needle < total[i]]
        kv[at] = 0.01
        kv[at, 0] = 40.0                                     # its normed latent is this direction and nothing else
    nw = torch.randn(rank, generator=g) * 0.1 + 1
    q, kv, uk, uv = (x.to(dtype) for x in (q, kv, uk, uv))
    f, want, r0 = lambda x: x.double(), [], 0
    for n, p0 in zip(total, past):
        rows = slice(r0, r0 + n)
        c = oracle.rms_norm(f(kv[rows, :rank]), eps, f(nw))
        turn = lambda x: oracle.rotate_pairs(x, rot, 1000.0)
        k = torch.cat([torch.einsum("hdr,tr->thd", f(uk), c), turn(f(kv[rows, None, rank:])).expand(n, heads, rot)], -1)
        qq = torch.cat([f(q[rows, :, :dim]), turn(f(q[rows, :, dim:]))], -1)
        want.append(oracle.causal_softmax_values(qq, k, torch.einsum("hdr,tr->thd", f(uv), c), sp.scale)[p0:])
        r0 += n
    pad = lambda x, n: torch.nn.functional.pad(x, (0, n - x.shape[-1]))
    rows = torch.cat([pad(q[:, :, :dim], sp.k_pad).reshape(n_all, -1), pad(q[:, :, dim:], sp.rot_pad).reshape(n_all, -1), pad(kv[:, :rank], sp.rank_pad),
                      pad(kv[:, rank:], sp.rot_pad)], -1)
    kv_up = torch.cat([torch.nn.functional.pad(w, (0, sp.rank_pad - rank, 0, p - w.shape[1])).reshape(heads * p, sp.rank_pad)
                       for w, p in ((uk, sp.k_pad), (uv, sp.v_pad))])
    key_up_t = kv_up[:heads * sp.k_pad].view(heads, sp.k_pad, sp.rank_pad).transpose(1, 2).contiguous()
    per = (max(total) + 63) // 64
    table = torch.randperm(per * len(lens) + 3, generator=g)[:per * len(lens)].reshape(len(lens), per).to(torch.int32)
    cache = (torch.randn(per * len(lens) + 3, 1, 1, 64, sp.pad, generator=g) * 3).to(dtype).to(device)     # leftovers of earlier requests
    cs = ops.rope_cos_sin(max(total), rot, 1000.0, None, device=device)
    starts = [sum(total[:i]) for i in range(len(lens))]
    dev = lambda x: x.to(device)

    def write(lo, hi):
        idx = torch.cat([torch.arange(s + a, s + b) for s, a, b in zip(starts, lo, hi)])
        meta = build_step_meta([b - a for a, b in zip(lo, hi)], lo, table, 64, device=device)
        return ops.latent_write(dev(rows[idx]), cache, meta, cs, dev(pad(nw, sp.rank_pad)), sp, eps), meta
    if any(past):
        write([0] * len(lens), past)
    x, meta = write(past, total)
    fn = ops.latent_attention if kernel is None else functools.partial(ops.cuda_ops().latent_attention, kernel=kernel)
    got = fn(x, cache, meta, dev(kv_up), dev(key_up_t), sp).float().cpu().view(-1, heads, sp.v_pad)
    assert sp.v_pad == dv or float(got[:, :, dv:].abs().max()) == 0.0
    w = torch.cat(want)
    if needle is not None:
        value = torch.einsum("hdr,r->hd", f(uv), oracle.rms_norm(f(kv[needle, :rank]), eps, f(nw)))
        seen = torch.cat([torch.arange(p0, n) >= needle for n, p0 in zip(total, past)])
        assert (w[seen] - value).abs().max() < 0.1 and (not (~seen).any() or (w[~seen] - value).abs().amax((1, 2)).min() > 0.5)
    return _worst_row(got[:, :, :dv].double() - w, w)


def _worst_row(d, w):
    """Largest root mean square of a (row, head) difference over the scale of the values."""
    return float(d.pow(2).mean(-1).sqrt().max() / w.std())


def unit_case(device, dtype, hq, hkv, d, dv, lens, past, coef, every, loud=None):
    """A step of :func:`ops.unit_kv_write` + :func:`ops.paged_attention`.  ``loud``: a position whose key points along every query."""
    from tensorrt_edge_llm_b200 import ops
    from tensorrt_edge_llm_b200.config import AttentionConfig
    from tensorrt_edge_llm_b200.ops.meta import build_step_meta
    sp = AttentionConfig(hq, hkv, d, dv, 0, scale=2.0 * d ** -0.5)
    g = torch.Generator().manual_seed(5)
    total, eps = [a + b for a, b in zip(lens, past)], 1e-4
    n_all = sum(total)
    q, k, v = torch.randn(n_all, hq, d, generator=g), torch.randn(n_all, hkv, d, generator=g), torch.randn(n_all, hkv, dv, generator=g)
    if loud is not None:
        q[:, :, 0] = 3.0 * d ** 0.5
        k[:, :, 0] = 0.0
        at = [sum(total[:i]) + loud for i in range(len(lens)) if loud < total[i]]
        k[at] = 0.0
        k[at, :, 0] = 1e-1                                  # small: only its direction counts
    q, k, v = (x.to(dtype) for x in (q, k, v))
    want, r0 = [], 0
    for n, p0 in zip(total, past):
        rows = slice(r0, r0 + n)
        qq = oracle.rms_norm(q[rows].double(), eps) * oracle.query_temperature(n, coef, every)[:, None, None]
        want.append(oracle.causal_softmax_values(qq, oracle.rms_norm(k[rows].double(), eps), v[rows].double(), sp.scale)[p0:])
        r0 += n
    pad = lambda x: torch.nn.functional.pad(x, (0, sp.pad - x.shape[-1])).reshape(n_all, -1)
    rows = torch.cat([pad(q), pad(k), pad(v)], -1)
    per = (max(total) + 63) // 64
    table = torch.randperm(per * len(lens) + 2, generator=g)[:per * len(lens)].reshape(len(lens), per).to(torch.int32)
    cache = torch.randn(per * len(lens) + 2, 2, hkv, 64, sp.pad, generator=g).to(dtype).to(device)
    temp = ops.query_temperature(max(total), coef, every, device)
    starts = [sum(total[:i]) for i in range(len(lens))]
    for lo, hi in (([0] * len(lens), past), (past, total)):
        if not any(hi):
            continue
        idx = torch.cat([torch.arange(s + a, s + b) for s, a, b in zip(starts, lo, hi)])
        meta = build_step_meta([b - a for a, b in zip(lo, hi)], lo, table, 64, device=device)
        qn = ops.unit_kv_write(rows[idx].to(device), cache, meta, temp, hq, hkv, sp.pad, d, eps)
    got = ops.paged_attention(qn, cache, meta, sp.scale, fp32_weights=True).float().cpu()
    w = torch.cat(want)
    if loud is not None:
        seen = torch.cat([torch.arange(p0, n) >= loud for n, p0 in zip(total, past)])
        assert seen.any()
    return _worst_row(got[:, :, :dv].double() - w, w)
