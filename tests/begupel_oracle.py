"""Plain, slow statement of the Begupel design in float64, one function per mechanism.

A whole sequence at a time, no cache, no batching, no kernels and nothing shared with the package: the tests compare the
framework against these loops.  ``cfg`` is the parsed ``config.json``, ``w`` maps checkpoint tensor names to tensors.
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, eps, gain=1.0):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def group_norm(x, gain, groups, eps):
    """Every one of ``groups`` equal parts of a row over its own root mean square."""
    parts = x.reshape(x.shape[0], groups, -1)
    return rms_norm(parts, eps).reshape(x.shape) * gain


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x):
    return x * torch.sigmoid(x)


def causal_conv(x, taps):
    """Depthwise convolution over time; the last tap multiplies the current row, rows before the start are zero."""
    n = taps.shape[1]
    out = torch.zeros_like(x)
    for j in range(n):
        back = n - 1 - j
        if back < x.shape[0]:
            out[back:] += taps[:, j] * x[:x.shape[0] - back]
    return out


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table per position; a sequence's first token takes the extra row behind the buckets."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + t * mul_cur) % buckets for i, t in enumerate(tokens)]


def embed(cfg, w, tokens):
    b = cfg["embedding"]["bigram"]
    rows = bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])
    return w["embed"][torch.as_tensor(tokens)] + w["bigram"][torch.as_tensor(rows)]


# ---- decayed outer-product memory ----------------------------------------------------------------------------


def decayed_memory(q, k, v, decay):
    """``S <- decay S + k v^T``, read by ``q`` after the write; ``q``, ``k`` ``[T, H, D]``, ``v`` ``[T, H, DV]``, ``decay`` ``[H]``."""
    s = torch.zeros(k.shape[1], k.shape[2], v.shape[2], dtype=F64)
    out = torch.zeros(v.shape, dtype=F64)
    for t in range(k.shape[0]):
        s = decay[:, None, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", s, q[t])
    return out


def lightning(h, c, w, p, eps):
    t, n = h.shape[0], c["heads"]
    q, k, v = (silu(h @ w[f"{p}.{m}"].T).reshape(t, n, -1) for m in "qkv")
    o = decayed_memory(q, k, v, torch.tensor(c["decay"], dtype=F64)).reshape(t, -1)
    return (rms_norm(o, eps, w[p + ".norm"]) * torch.sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


# ---- attention with rotated values ---------------------------------------------------------------------------


def turn(x, dims, base, factor=1.0, back=False):
    """Rotation by position of the first ``dims`` features of ``x`` ``[T, H, D]``, neighbours forming the pairs; ``back``: the other way."""
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=F64)[:, None] * (-1.0 if back else 1.0)
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims) / factor
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[:, :, 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def window_softmax_values(q, k, v, scale, window):
    """``q`` ``[T, H, D]``, ``k`` ``[T, G, D]``, ``v`` ``[T, G, DV]``; query head ``n`` reads key head ``n // (H // G)``; a row sees itself and
    the ``window - 1`` rows before it."""
    t, heads, group = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    gap = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    hidden = (gap < 0) | (gap >= window)
    out = torch.zeros(t, heads, v.shape[2], dtype=F64)
    for n in range(heads):
        s = (q[:, n] @ k[:, n // group].T) * scale
        out[:, n] = torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, n // group]
    return out


def attention_heads(q, k, v, c):
    """Heads of queries, keys (normed, not yet rotated) and values: the outputs before the output projection."""
    rot, dv = c["rot"], v.shape[2]
    q, k = (turn(x, rot["dims"], rot["base"], rot["scaling"]["factor"]) for x in (q, k))
    o = window_softmax_values(q, k, turn(v, dv, rot["base"]), c["scale"], c["mask"]["size"])
    return turn(o, dv, rot["base"], back=True)


def attention(h, c, w, p, eps):
    t, n, g = h.shape[0], c["heads"], c["kv_heads"]
    q = rms_norm(h @ w[p + ".q"].T, eps, w[p + ".q.norm"]).reshape(t, n, -1)
    k = rms_norm(h @ w[p + ".k"].T, eps, w[p + ".k.norm"]).reshape(t, g, -1)
    v = (h @ w[p + ".v"].T).reshape(t, g, -1)
    return attention_heads(q, k, v, c).reshape(t, -1) @ w[p + ".o"].T


# ---- gated delta rule ----------------------------------------------------------------------------------------


def delta_recurrence(q, k, v, g, beta):
    """Delta rule with one decay per head; ``q``, ``k`` ``[T, H, D]``, ``v`` ``[T, H, DV]``, ``g``, ``beta`` ``[T, H]``."""
    s = torch.zeros(k.shape[1], k.shape[2], v.shape[2], dtype=F64)
    out = torch.zeros(v.shape, dtype=F64)
    for t in range(k.shape[0]):
        s = g[t][:, None, None] * s
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", s, k[t]))
        s = s + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", s, q[t])
    return out


def head_decay(z, a_log, bias):
    return torch.exp(-torch.exp(a_log) * torch.nn.functional.softplus(z + bias, threshold=700.0))


def delta_rule(h, c, w, p, eps):
    t, n, kv, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q, k, v = (silu(causal_conv(h @ w[f"{p}.{m}"].T, w[f"{p}.{m}.conv"])) for m in "qkv")
    rep = n // kv
    q = (unit(q.reshape(t, kv, d)) * d ** -0.5).repeat_interleave(rep, 1)
    k = unit(k.reshape(t, kv, d)).repeat_interleave(rep, 1)
    beta, g = torch.sigmoid(h @ w[p + ".b"].T), head_decay(h @ w[p + ".a"].T, w[p + ".A_log"], w[p + ".dt_bias"])
    o = rms_norm(delta_recurrence(q, k, v.reshape(t, n, -1), g, beta), eps, w[p + ".norm"]).reshape(t, -1)
    return (o * silu(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def parallel(h, c, w, p, eps):
    return c["left_scale"] * attention(h, c["left"], w, p + ".left", eps) + c["right_scale"] * delta_rule(h, c["right"], w, p + ".right", eps)


# ---- layers and model ----------------------------------------------------------------------------------------


def dense(h, w, p):
    gate, up = (h @ w[f"{p}.{m}"].T + w[f"{p}.{m}.b"] for m in ("gate", "up"))
    return (torch.relu(gate) * up) @ w[p + ".down"].T + w[p + ".down.b"]


MIXERS = {"lightning": lightning, "parallel": parallel}


def layer(x, c, w, name, norm):
    groups, eps = norm["groups"], norm["eps"]
    h = x + causal_conv(x, w[name + ".canon1"])
    x = x + group_norm(MIXERS[c["type"]](h, c["mixer"], w, name + ".mix", eps), w[name + ".norm1"], groups, eps)
    if c.get("mlp"):
        x = x + group_norm(dense(x, w, name + ".mlp"), w[name + ".norm2"], groups, eps)
    return x


def softcap(x, cap):
    return cap * torch.tanh(x / cap)


def forward(cfg, w, tokens, trace=None):
    """Logits ``[T, vocab]``; ``trace`` (a list) collects the residual stream after every layer."""
    w = {k: v.to(F64) for k, v in w.items()}
    x = embed(cfg, w, [int(t) for t in tokens])
    for i, c in enumerate(cfg["layers"]):
        x = layer(x, c, w, f"l{i}", cfg["norm"])
        if trace is not None:
            trace.append(x)
    h = group_norm(x, w["final.norm"], cfg["norm"]["groups"], cfg["norm"]["eps"])
    return softcap(h @ w["head"].T, cfg["logit_softcap"])


def greedy(cfg, w, prompt, steps):
    """Greedy continuation by recomputing the whole sequence for every token."""
    toks = list(prompt)
    for _ in range(steps):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
