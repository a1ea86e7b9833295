"""Plain, slow statement of the Dimesun design in float64, one function per mechanism.

A whole sequence at a time, no cache, no batching, no kernels and nothing shared with the package: the tests compare the
framework against these loops.  ``cfg`` is the parsed ``config.json``, ``w`` maps checkpoint tensor names to tensors.
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, gain, eps):
    """Rows of ``x`` over their root mean square, times ``gain``."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def rotate(x, positions, dims, base):
    """Rotate-half rotary positions on the first ``dims`` features of ``x`` ``[T, H, D]``."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        angle = positions.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def chunk_visible(i, j, size):
    """Whether position ``i`` sees position ``j`` under a chunked causal mask (``size`` 0 = plain causal)."""
    return j <= i and (not size or i // size == j // size)


def sink_softmax(scores):
    """Softmax whose denominator holds one more term, exp(0), that belongs to no key."""
    m = max(0.0, float(scores.max()))
    e = torch.exp(scores - m)
    return e / (math.exp(-m) + e.sum())


def attention(h, c, w, p):
    """Chunked attention with grouped heads, partial rotary and a zero sink.  ``h`` ``[T, width]``."""
    t, heads, kv, d, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = (h @ w[p + ".q"].T).reshape(t, heads, d)
    k = (h @ w[p + ".k"].T).reshape(t, kv, d)
    v = (h @ w[p + ".v"].T).reshape(t, kv, dv)
    pos = torch.arange(t)
    q = rotate(q, pos, c["rot"]["dims"], c["rot"]["base"])
    k = rotate(k, pos, c["rot"]["dims"], c["rot"]["base"])
    size = c["mask"]["size"]
    out = torch.zeros(t, heads, dv, dtype=F64)
    for i in range(t):
        seen = [j for j in range(i + 1) if chunk_visible(i, j, size)]
        for n in range(heads):
            g = n // (heads // kv)
            s = (k[seen, g] @ q[i, n]) * c["scale"]
            out[i, n] = sink_softmax(s) @ v[seen, g]
    return out.reshape(t, heads * dv) @ w[p + ".o"].T


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def mlstm_recurrence(q, k, v, log_i, log_f):
    """Matrix memory with a running maximum, one head: ``q``, ``k`` ``[T, D]``, ``v`` ``[T, DV]``, gates ``[T]``."""
    t, d = k.shape
    s = torch.zeros(d, v.shape[1], dtype=F64)
    n = torch.zeros(d, dtype=F64)
    m = 0.0
    out = torch.zeros(t, v.shape[1], dtype=F64)
    for i in range(t):
        m_new = max(float(log_f[i]) + m, float(log_i[i]))
        keep, add = math.exp(float(log_f[i]) + m - m_new), math.exp(float(log_i[i]) - m_new)
        s = keep * s + add * torch.outer(k[i], v[i])
        n = keep * n + add * k[i]
        m = m_new
        out[i] = (s.T @ q[i]) / (max(abs(float(n @ q[i])), math.exp(-m)) + 1e-6)
    return out


def mlstm(h, c, w, p, eps):
    t, heads, d, dv, cap = h.shape[0], c["heads"], c["dim"], c["vdim"], c["gate_cap"]
    q = (h @ w[p + ".q"].T).reshape(t, heads, d) * d ** -0.5
    k = (h @ w[p + ".k"].T).reshape(t, heads, d)
    v = (h @ w[p + ".v"].T).reshape(t, heads, dv)
    log_i = soft_cap(h @ w[p + ".i"].T + w[p + ".i.b"], cap)
    log_f = torch.nn.functional.logsigmoid(soft_cap(h @ w[p + ".f"].T + w[p + ".f.b"], cap))
    o = torch.stack([mlstm_recurrence(q[:, n], k[:, n], v[:, n], log_i[:, n], log_f[:, n]) for n in range(heads)], dim=1)
    o = rms_norm(o, 1.0, eps).reshape(t, heads * dv) * w[p + ".norm"]
    return (o * torch.sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def clamped_glu(gate, up, limit):
    g, u = torch.clamp(gate, max=limit), torch.clamp(up, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def route(z, top):
    """Indices of the ``top`` largest logits and the softmax over them."""
    val, idx = torch.topk(z, top)
    return idx, torch.softmax(val, -1)


def experts(h, c, w, p):
    limit, top = c["expert"]["limit"], c["router"]["top"]
    z = h @ w[p + ".router"].T + w[p + ".router.b"]
    out = torch.zeros_like(h)
    for i in range(h.shape[0]):
        idx, wt = route(z[i], top)
        for e, a in zip(idx.tolist(), wt):
            y = clamped_glu(w[f"{p}.e{e}.gate"] @ h[i], w[f"{p}.e{e}.up"] @ h[i], limit)
            out[i] += a * (w[f"{p}.e{e}.down"] @ y)
    return out


def layer(x, c, w, name, eps, mult):
    h = rms_norm(x, 1 + w[name + ".norm1"], eps)
    y = attention(h, c["mixer"], w, name + ".mix") if c["type"] == "attention" else mlstm(h, c["mixer"], w, name + ".mix", eps)
    if c.get("mlp"):
        y = y + experts(h, c["mlp"], w, name + ".mlp")
    return x + mult * y


def schedule(cfg):
    """The layer runs in order: ``(layer, pass or None, whether it is the first layer of its pass)``."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None, False) for i in range(n)]
    runs = [(i, None, False) for i in range(lp["start"])]
    for t in range(lp["times"]):
        runs += [(i, t, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return runs + [(i, None, False) for i in range(lp["stop"], n)]


def forward(cfg, w, tokens, trace=None):
    """Logits ``[T, vocab]``; ``trace`` (a list) collects the residual stream after every layer run."""
    w = {k: v.to(F64) for k, v in w.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens)]
    for i, t, first in schedule(cfg):
        if first:
            x = x + w["loop.step"][t]
        x = layer(x, cfg["layers"][i], w, f"l{i}", eps, mult)
        if trace is not None:
            trace.append(x)
    return rms_norm(x, 1 + w["final.norm"], eps) @ w["embed"].T


def greedy(cfg, w, prompt, steps):
    """Greedy continuation by recomputing the whole sequence for every token."""
    toks = list(prompt)
    for _ in range(steps):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def small_config(layers, width=64, vocab=96, loop=None, eps=1e-5, mult=0.5):
    """A ``config.json`` dictionary.  ``layers``: ``(type, mixer, mlp)`` triples."""
    cfg = {"architecture": "Dimesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
           "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in layers]}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def attn_mixer(heads, kv, dim, vdim=None, size=32, rot=None, base=10000.0, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim or dim, "mask": {"size": size},
            "rot": {"dims": rot or dim, "base": base}, "scale": scale or dim ** -0.5}


def mlstm_mixer(heads, dim, vdim=None, cap=15.0):
    return {"heads": heads, "dim": dim, "vdim": vdim or dim, "gate_cap": cap}


def moe(experts=6, top=2, ff=32, limit=7.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def random_weights(cfg, seed=0, gain=1.0):
    """bfloat16 tensors of every name the design has; scaled so that activations stay near one."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s * gain / math.sqrt(i))).bfloat16()

    def vec(n, s, off=0.0):
        return (torch.randn(n, generator=g) * s + off).bfloat16()
    d = cfg["width"]
    w = {"embed": torch.randn(cfg["vocab"], d, generator=g).bfloat16(), "final.norm": vec(d, 0.2)}
    if cfg.get("loop"):
        w["loop.step"] = (torch.randn(cfg["loop"]["times"], d, generator=g) * 0.3).bfloat16()
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}"
        w[p + ".norm1"] = vec(d, 0.2)
        kv = m.get("kv_heads", m["heads"])
        w[p + ".mix.q"] = mat(m["heads"] * m["dim"], d, 1.5)
        w[p + ".mix.k"] = mat(kv * m["dim"], d, 1.5)
        w[p + ".mix.v"] = mat(kv * m["vdim"], d)
        w[p + ".mix.o"] = mat(d, m["heads"] * m["vdim"], 2.0)
        if l["type"] == "mlstm":
            w[p + ".mix.g"] = mat(m["heads"] * m["vdim"], d)
            w[p + ".mix.norm"] = vec(m["heads"] * m["vdim"], 0.2, 1.0)
            w[p + ".mix.i"], w[p + ".mix.i.b"] = mat(m["heads"], d, 2.0), vec(m["heads"], 1.0)
            w[p + ".mix.f"], w[p + ".mix.f.b"] = mat(m["heads"], d, 2.0), vec(m["heads"], 1.0, 3.0)
        if l.get("mlp"):
            f = l["mlp"]
            w[p + ".mlp.router"], w[p + ".mlp.router.b"] = mat(f["router"]["experts"], d, 2.0), vec(f["router"]["experts"], 0.5)
            for e in range(f["router"]["experts"]):
                w[f"{p}.mlp.e{e}.gate"], w[f"{p}.mlp.e{e}.up"] = mat(f["expert"]["ff"], d), mat(f["expert"]["ff"], d)
                w[f"{p}.mlp.e{e}.down"] = mat(d, f["expert"]["ff"], 2.0)
    return w
