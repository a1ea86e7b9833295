"""Plain, slow statement of the Debonex design in float64, one function per mechanism.

A whole sequence at a time, no cache, no batching, no kernels and nothing shared with the package: the tests compare the
framework against these loops.  ``cfg`` is the parsed ``config.json``, ``w`` maps checkpoint tensor names to tensors.
"""
import math

import torch

F64 = torch.float64


def dynamic_tanh(x, w, name):
    """Element-wise norm: no statistics, a squashed row with gain and shift."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rms_norm(x, eps, gain=1.0):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def short_conv(x, taps):
    """Causal depthwise convolution over time; the last tap multiplies the current row."""
    n = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            src = t - (n - 1 - j)
            if src >= 0:
                out[t] += taps[:, j] * x[src]
    return out


def delta_recurrence(q, k, v, g, beta):
    """Delta rule with one decay per key channel, one head: ``q``, ``k``, ``g`` ``[T, D]``, ``v`` ``[T, DV]``, ``beta`` ``[T]``."""
    s = torch.zeros(k.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros(v.shape, dtype=F64)
    for t in range(k.shape[0]):
        s = g[t][:, None] * s
        u = beta[t] * (v[t] - s.T @ k[t])
        s = s + torch.outer(k[t], u)
        out[t] = s.T @ q[t]
    return out


def channel_decay(h, w, p, heads, dim):
    """``[T, heads, dim]`` factors in (0, 1)."""
    z = (h @ w[p + ".a1"].T) @ w[p + ".a2"].T + w[p + ".dt_bias"]
    soft = torch.nn.functional.softplus(z, threshold=700.0).reshape(-1, heads, dim)
    return torch.exp(-torch.exp(w[p + ".A_log"])[:, None] * soft)


def channel_delta(h, c, w, p, eps):
    t, heads, kv, d, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(short_conv(h @ w[f"{p}.{n}"].T, w[f"{p}.{n}.conv"])) for n in "qkv")
    q, k, v = unit(q.reshape(t, kv, d)) * d ** -0.5, unit(k.reshape(t, kv, d)), v.reshape(t, heads, dv)
    beta, g = torch.sigmoid(h @ w[p + ".b"].T), channel_decay(h, w, p, heads, d)
    o = torch.stack([delta_recurrence(q[:, n // (heads // kv)], k[:, n // (heads // kv)], v[:, n], g[:, n], beta[:, n])
                     for n in range(heads)], dim=1)
    o = rms_norm(o, eps, w[p + ".norm"]).reshape(t, heads * dv)
    return (o * torch.sigmoid((h @ w[p + ".g1"].T) @ w[p + ".g2"].T)) @ w[p + ".o"].T


def rotate_pairs(x, dims, base):
    """Rotation by position on the first ``dims`` features of ``x`` ``[T, H, D]``, neighbours forming the pairs."""
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=F64)[:, None]
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[:, :, 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def causal_softmax_values(q, k, v, scale):
    """``q`` ``[T, H, D]``, ``k`` ``[T, G, D]``, ``v`` ``[T, G, DV]``; query head ``n`` reads key head ``n // (H // G)``."""
    t, heads, group = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    hidden = torch.triu(torch.ones(t, t, dtype=torch.bool), 1)
    out = torch.zeros(t, heads, v.shape[2], dtype=F64)
    for n in range(heads):
        s = (q[:, n] @ k[:, n // group].T) * scale
        out[:, n] = torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, n // group]
    return out


def latent_attention(h, c, w, p, eps):
    t, heads, d, r, dv, rank = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    q = (h @ w[p + ".q"].T).reshape(t, heads, d + r)
    kv = h @ w[p + ".dkv"].T
    c_kv = rms_norm(kv[:, :rank], eps, w[p + ".dkv.norm"])
    k = (c_kv @ w[p + ".uk"].T).reshape(t, heads, d)
    v = (c_kv @ w[p + ".uv"].T).reshape(t, heads, dv)
    turn = lambda x: rotate_pairs(x, c["rot"]["dims"], c["rot"]["base"])
    k_rot = turn(kv[:, None, rank:]).expand(t, heads, r)
    q = torch.cat((q[:, :, :d], turn(q[:, :, d:])), -1)
    o = causal_softmax_values(q, torch.cat((k, k_rot), -1), v, c["scale"])
    return o.reshape(t, heads * dv) @ w[p + ".o"].T


def query_temperature(t, coef, every):
    """``[T]`` factors that grow with the logarithm of the position's block."""
    return torch.tensor([1 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(t)], dtype=F64)


def attention(h, c, w, p, eps):
    t, heads, kv, d, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rms_norm((h @ w[p + ".q"].T).reshape(t, heads, d), eps)
    k = rms_norm((h @ w[p + ".k"].T).reshape(t, kv, d), eps)
    v = (h @ w[p + ".v"].T).reshape(t, kv, dv)
    if c.get("q_temp"):
        q = q * query_temperature(t, c["q_temp"]["coef"], c["q_temp"]["every"])[:, None, None]
    return causal_softmax_values(q, k, v, c["scale"]).reshape(t, heads * dv) @ w[p + ".o"].T


def dense(h, w, p):
    return (gelu_tanh(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


MIXERS = {"channel_delta": channel_delta, "latent_attention": latent_attention, "attention": attention}


def layer(x, c, w, name, eps):
    x = x + MIXERS[c["type"]](dynamic_tanh(x, w, name + ".norm1"), c["mixer"], w, name + ".mix", eps)
    if c.get("mlp"):
        x = x + dense(dynamic_tanh(x, w, name + ".norm2"), w, name + ".mlp")
    return x


def forward(cfg, w, tokens, trace=None):
    """Logits ``[T, vocab]``; ``trace`` (a list) collects the residual stream after every layer."""
    w = {k: v.to(F64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, c in enumerate(cfg["layers"]):
        x = layer(x, c, w, f"l{i}", eps)
        if trace is not None:
            trace.append(x)
    return dynamic_tanh(x, w, "final.norm") @ w["head"].T * cfg["logit_scale"]


def greedy(cfg, w, prompt, steps):
    """Greedy continuation by recomputing the whole sequence for every token."""
    toks = list(prompt)
    for _ in range(steps):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def small_config(layers, width=64, vocab=96, eps=1e-5, emb=2.0, logit_scale=1.5):
    """A ``config.json`` dictionary.  ``layers``: ``(type, mixer, ff or None)`` triples."""
    return {"architecture": "Debonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": emb},
            "logit_scale": logit_scale,
            "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": f} if f else None} for t, m, f in layers]}


def delta_mixer(heads, kv, dim, vdim, conv=4):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def latent_mixer(heads, dim, rot_dim, vdim, rank, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "rot": {"dims": rot_dim, "base": base},
            "scale": scale or (dim + rot_dim) ** -0.5}


def attn_mixer(heads, kv, dim, vdim, coef=0.3, every=50, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "q_temp": {"coef": coef, "every": every}}


def random_weights(cfg, seed=0, rank_a=8, rank_g=12):
    """bfloat16 tensors of every name the design has; scaled so that activations stay near one."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s / math.sqrt(i))).bfloat16()

    def vec(n, s, off=0.0):
        return (torch.randn(n, generator=g) * s + off).bfloat16()
    d = cfg["width"]
    w = {"embed": mat(cfg["vocab"], d, d ** 0.5 / cfg["embedding"]["scale"]), "head": mat(cfg["vocab"], d)}

    def norm(name):
        w[name], w[name + ".b"], w[name + ".alpha"] = vec(d, 0.2, 1.0), vec(d, 0.2), vec(1, 0.1, 0.7).reshape(())
    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix"
        norm(f"l{i}.norm1")
        h, dim, dv = m["heads"], m["dim"], m["vdim"]
        if l["type"] == "latent_attention":
            r, rank = m["rot_dim"], m["kv_rank"]
            w[p + ".q"], w[p + ".dkv"], w[p + ".dkv.norm"] = mat(h * (dim + r), d, 2.0), mat(rank + r, d, 2.0), vec(rank, 0.2, 1.0)
            w[p + ".uk"], w[p + ".uv"] = mat(h * dim, rank), mat(h * dv, rank)
        else:
            kv = m["kv_heads"]
            w[p + ".q"], w[p + ".k"], w[p + ".v"] = mat(kv * dim if l["type"] == "channel_delta" else h * dim, d), mat(kv * dim, d), None
            w[p + ".v"] = mat(h * dv if l["type"] == "channel_delta" else kv * dv, d, 1.5)
        if l["type"] == "channel_delta":
            for n in "qkv":
                w[f"{p}.{n}.conv"] = (torch.randn(w[f"{p}.{n}"].shape[0], m["conv"], generator=g) * 0.6).bfloat16()
            w[p + ".b"], w[p + ".A_log"], w[p + ".norm"] = mat(h, d, 1.5), vec(h, 0.5, 0.5), vec(dv, 0.2, 1.0)
            w[p + ".a1"], w[p + ".a2"], w[p + ".dt_bias"] = mat(rank_a, d), mat(h * dim, rank_a, 1.5), vec(h * dim, 1.5, -3.5)
            w[p + ".g1"], w[p + ".g2"] = mat(rank_g, d), mat(h * dv, rank_g, 1.5)
        w[p + ".o"] = mat(d, h * dv, 1.5)
        if l.get("mlp"):
            f = l["mlp"]["ff"]
            norm(f"l{i}.norm2")
            w[f"l{i}.mlp.gate"], w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"] = mat(f, d, 1.5), mat(f, d, 1.5), mat(d, f, 1.5)
    return w
