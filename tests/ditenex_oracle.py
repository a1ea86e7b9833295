"""Plain, slow statement of the Ditenex design in float64, one function per mechanism.

A whole sequence at a time, no cache, no batching, no kernels and nothing shared with the package: the tests compare the
framework against these loops.  ``cfg`` is the parsed ``config.json``, ``w`` maps checkpoint tensor names to tensors.
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, eps, gain=1.0):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def embed(w, tokens):
    """Token row plus the row of the position, both learned."""
    return w["embed"][torch.as_tensor(tokens)] + w["pos"][:len(tokens)]


def token_shift(h, amount):
    """Every feature moves by its own share towards the row before it (zeros in front of the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * amount


# ---- attention with mixed scores -----------------------------------------------------------------------------


def distance_slopes(heads):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=F64)


def head_scores(q, k, scale):
    """``[H, T, T]`` scores of ``q`` ``[T, H, D]`` and ``k`` ``[T, G, D]``: dot products times ``scale``, less slope times distance."""
    t, heads, group = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    gap = (torch.arange(t)[:, None] - torch.arange(t)[None, :]).to(F64)
    slope = distance_slopes(heads)
    return torch.stack([(q[:, n] @ k[:, n // group].T) * scale - slope[n] * gap for n in range(heads)])


def mix_heads(s, talk):
    """Score of head ``n``: the sum of all heads' scores with the weights of row ``n``."""
    out = torch.zeros_like(s)
    for n in range(s.shape[0]):
        for g in range(s.shape[0]):
            out[n] += talk[n, g] * s[g]
    return out


def window_weights(s, window):
    """Softmax over the row's own key and the ``window - 1`` keys before it."""
    t = s.shape[1]
    gap = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return torch.softmax(s.masked_fill((gap < 0) | (gap >= window), -math.inf), -1)


def attend(q, k, v, talk, scale, window):
    """Heads ``[T, H, DV]``; query head ``n`` reads value head ``n // (H // G)``."""
    a = window_weights(mix_heads(head_scores(q, k, scale), talk), window)
    group = q.shape[1] // v.shape[1]
    return torch.stack([a[n] @ v[:, n // group] for n in range(q.shape[1])], 1)


def mix_values(v, first, share):
    return (1.0 - share) * v + share * first


def attention(h, c, w, p, first):
    """``(output, values of the first layer that mixes)``; ``first`` is None until that layer has run."""
    t, n, g = h.shape[0], c["heads"], c["kv_heads"]
    q, k, v = (h @ w[f"{p}.{m}"].T + w[f"{p}.{m}.b"] for m in "qkv")
    if c["v_mix"]:
        if first is None:
            first = v
        else:
            v = mix_values(v, first, w[p + ".vmix"])
    o = attend(q.reshape(t, n, -1), k.reshape(t, g, -1), v.reshape(t, g, -1), w[p + ".talk"], c["scale"], c["mask"]["size"])
    return (o.reshape(t, -1) * torch.sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T, first


# ---- feed-forwards -------------------------------------------------------------------------------------------


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp(min=0)


def xielu(z, p, q):
    """Quadratic above zero, exponential below, slope one half at zero."""
    neg = z.clamp(max=0)
    return torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(neg) - neg)) + z / 2


def dense(h, w, p):
    return xielu(h @ w[p + ".up"].T, w[p + ".act"][0], w[p + ".act"][1]) @ w[p + ".down"].T


def gated_unit(h, w, p):
    gate = h @ w[p + ".gate"].T
    return (gate * torch.sigmoid(gate) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def chosen_experts(choice, top, count, keep):
    """Experts of one token by their choice scores: the ``top`` best inside the ``keep`` best of ``count`` equal groups, a group judged by
    the sum of its two best."""
    groups = choice.reshape(count, -1)
    score = groups.topk(min(2, groups.shape[1]), -1).values.sum(-1)
    open_ = set(score.topk(keep).indices.tolist())
    size = groups.shape[1]
    order = sorted((e for e in range(choice.shape[0]) if e // size in open_), key=lambda e: -float(choice[e]))
    return order[:top]


def routed(h, c, w, p):
    r = c["router"]
    scores = torch.sigmoid(h @ w[p + ".router"].T)
    choice = scores + w[p + ".correction"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in chosen_experts(choice[t], r["top"], r["groups"]["count"], r["groups"]["keep"]):
            out[t] += scores[t, e] * r["scale"] * gated_unit(h[t], w, f"{p}.e{e}")
    return out


def feed_forward(h, c, w, p):
    if c["kind"] == "dense":
        return dense(h, w, p)
    out = routed(h, c, w, p)
    return out + gated_unit(h, w, p + ".shared") if c.get("shared") else out


# ---- layers and model ----------------------------------------------------------------------------------------


def layer(x, c, w, name, eps, mult, first):
    h = token_shift(rms_norm(x, eps, w[name + ".norm1"]), w[name + ".shift"])
    y, first = attention(h, c["mixer"], w, name + ".mix", first)
    x = x + mult * rms_norm(y, eps, w[name + ".norm1b"])
    if c.get("mlp"):
        y = feed_forward(rms_norm(x, eps, w[name + ".norm2"]), c["mlp"], w, name + ".mlp")
        x = x + mult * rms_norm(y, eps, w[name + ".norm2b"])
    return x, first


def forward(cfg, w, tokens, trace=None):
    """Logits ``[T, vocab]``; ``trace`` (a list) collects the residual stream after every layer."""
    w = {k: v.to(F64) for k, v in w.items()}
    eps, first = cfg["norm"]["eps"], None
    x = embed(w, [int(t) for t in tokens])
    for i, c in enumerate(cfg["layers"]):
        x, first = layer(x, c, w, f"l{i}", eps, cfg["residual_mult"], first)
        if trace is not None:
            trace.append(x)
    return rms_norm(x, eps, w["final.norm"]) @ w["embed"].T


def greedy(cfg, w, prompt, steps):
    """Greedy continuation by recomputing the whole sequence for every token."""
    toks = list(prompt)
    for _ in range(steps):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
