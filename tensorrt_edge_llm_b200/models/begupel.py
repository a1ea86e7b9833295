"""Begupel decoder: layers listed one by one over an fp32 residual stream, normed behind every sublayer instead of in front of it.

``h = x + conv(x)`` (a short causal convolution over time), ``x += norm1(mixer(h))``, then ``x += norm2(mlp(x))``; the norm divides equal parts
of a row by their own root mean square.  The mixer is lightning attention, or windowed attention with rotated values beside a
gated delta rule; the feed-forward is a relu-gated unit with biases (or absent).  Embeddings are the sum of a token row and a row of
a bigram table; logits are capped.

Between two sublayers one kernel (``ops.stream_post``) norms the sublayer's output, adds it to the stream and writes what the next one
reads: the stream itself for a feed-forward, the convolved stream for a mixer, the final norm for the head.  The convolution's history
(rows of the stream, fp32) and the last token of a sequence are state rows indexed by seat.
"""
from __future__ import annotations

import re
from typing import Dict, Optional

import torch
from torch import nn

from .. import ops
from ..config import LAYER_LIGHTNING, LAYER_PARALLEL, ModelConfig
from ..model import register_model
from ..ops.meta import StepMeta
from .default import GatedMLP
from .linear import Fp32OutLinear
from .nemotron_h import HybridCausalLM, LightningMixer, ParallelMixer


class PartNorm(nn.Module):
    """Weight of an RMS norm over equal parts of a row; applied by ``ops.stream_post``."""

    def __init__(self, dim: int):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(dim, dtype=torch.float32), requires_grad=False)


class InputConv(nn.Module):
    """Taps of the depthwise causal convolution in front of a mixer, one row per tap (the last one multiplies the current row)."""

    def __init__(self, dim: int, taps: int, prefix: str):
        super().__init__()
        self.prefix = prefix
        self.weight = nn.Parameter(torch.zeros(taps, dim, dtype=torch.float32), requires_grad=False)

    @torch.no_grad()
    def load_checkpoint(self, fetch) -> bool:
        w = fetch(f"{self.prefix}.taps")
        if w is not None:
            self.weight.copy_(w.float().t())
        return False

    @torch.no_grad()
    def random_init(self, gen, std=0.02):
        self.weight.copy_(torch.randn(self.weight.shape, generator=gen) * 0.2)


class BegupelLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, idx: int):
        super().__init__()
        spec, p = cfg.layer_specs[idx], f"model.layers.{idx}"
        self.kind, self.spec, self.idx = spec.kind, spec, idx
        self.conv = InputConv(cfg.hidden_size, cfg.input_conv, f"{p}.conv")
        self.mixer = (ParallelMixer if spec.kind == LAYER_PARALLEL else LightningMixer)(cfg, spec if spec.kind == LAYER_PARALLEL else spec.lightning, f"{p}.mixer")
        self.norm = PartNorm(cfg.hidden_size)
        self.mlp = None
        if spec.ff:
            self.mlp_norm = PartNorm(cfg.hidden_size)
            self.mlp = GatedMLP(cfg, spec.ff, act=spec.ff_act, bias=spec.ff_bias)

    def mix(self, h: torch.Tensor, meta: StepMeta, cache, table):
        """``(output, sums of the row behind it that it still has to be divided by, or None)``."""
        if self.kind == LAYER_LIGHTNING:
            return self.mixer(h, meta, cache.recurrent, self.idx)
        return self.mixer(h, meta, cache, table, self.idx), None


class BegupelTransformer(nn.Module):
    def __init__(self, cfg: ModelConfig):
        super().__init__()
        self.cfg = cfg
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=cfg.compute_dtype)
        self.embed_tokens.weight.requires_grad_(False)
        if cfg.bigram_buckets:
            self.embed_bigrams = nn.Embedding(cfg.bigram_buckets + 1, cfg.hidden_size, dtype=cfg.compute_dtype)
            self.embed_bigrams.weight.requires_grad_(False)
        else:
            self.embed_bigrams = None
        self.layers = nn.ModuleList([BegupelLayer(cfg, i) for i in range(len(cfg.layer_specs))])
        self.norm = PartNorm(cfg.hidden_size)

    def source(self, ids, state) -> dict:
        """Arguments that make ``ops.stream_post`` start the stream from token ids."""
        cfg, out = self.cfg, dict(ids=ids, table=self.embed_tokens.weight)
        if self.embed_bigrams is not None:
            out["bigram"] = ops.Bigram(self.embed_bigrams.weight, state.tokens[0], cfg.bigram_buckets, cfg.bigram_mul_prev, cfg.bigram_mul_cur)
        return out

    def conv_args(self, i: int, state) -> dict:
        return dict(conv=self.layers[i].conv.weight, history=state.inputs.get(i))

    def forward(self, ids, meta, cache, tables, comm, inputs_embeds=None, capture_layers=()):
        if inputs_embeds is not None or hasattr(self.embed_tokens.weight, "lookup"):
            raise NotImplementedError("this family embeds pairs of tokens: it takes token ids and plain tables")
        cfg, state = self.cfg, cache.recurrent
        step = lambda x, y, w, **kw: ops.stream_post(x, y, None if w is None else w.weight, cfg.norm_groups, cfg.rms_norm_eps, meta, cfg.compute_dtype, **kw)
        rec = state.record
        if rec is not None:
            rec["ids"] = ids
        x, h = step(None, None, None, **self.source(ids, state), **self.conv_args(0, state))
        taps, last = [], len(self.layers) - 1
        for i, layer in enumerate(self.layers):
            (y, sums), norm = layer.mix(h, meta, cache, tables.get(i)), layer.norm
            if layer.mlp is not None:
                x, h = step(x, y, norm, sums=sums)
                y, sums, norm = layer.mlp(h), None, layer.mlp_norm
            x, h = step(x, y, norm, sums=sums, **(dict(out_norm=self.norm.weight) if i == last else self.conv_args(i + 1, state)))
            if rec is not None and i < last:
                rec["inputs", i + 1] = x
            if i in capture_layers:
                taps.append(x)
        return (h, taps) if capture_layers else h


@register_model("begupel")
class BegupelCausalLM(HybridCausalLM):
    transformer_cls = BegupelTransformer

    def __init__(self, cfg: ModelConfig, comm=None):
        if cfg.tp_size > 1 or cfg.mapping.ep_size > 1:
            raise NotImplementedError("tensor and expert parallelism are not built for the begupel family")
        if cfg.quant.is_quantized:
            raise NotImplementedError("quantised weights are not built for the begupel family")
        if cfg.hidden_size % 8:
            raise ValueError("the model width must be a multiple of 8")
        if cfg.dtype == "float16":
            raise ValueError("the begupel family runs in bfloat16 or float32: rows that no norm has scaled leave the range of float16")
        super().__init__(cfg, comm)
        self.lm_head = Fp32OutLinear(cfg.hidden_size, [cfg.vocab_size], dtype=cfg.compute_dtype)
        self._tables: Dict[tuple, torch.Tensor] = {}

    # ---- checkpoint names ---------------------------------------------------------------------------
    _MIX = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "g": "g_proj.weight", "o": "o_proj.weight", "b": "beta_proj.weight",
            "a": "decay_proj.weight", "q.norm": "q_norm.weight", "k.norm": "k_norm.weight", "q.conv": "q_conv", "k.conv": "k_conv", "v.conv": "v_conv",
            "A_log": "a_log", "norm": "head_norm.weight"}

    def checkpoint_key_remap(self, name: str) -> Optional[str]:
        flat = {"embed": "model.embed_tokens.weight", "bigram": "model.embed_bigrams.weight", "head": "lm_head.weight", "final.norm": "model.norm.weight"}
        if name in flat:
            return flat[name]
        m = re.fullmatch(r"l(\d+)\.(.+)", name)
        if not m:
            return name
        p, rest = f"model.layers.{m[1]}", m[2]
        fixed = {"norm1": "norm.weight", "norm2": "mlp_norm.weight", "canon1": "conv.taps"}
        if rest in fixed:
            return f"{p}.{fixed[rest]}"
        f = re.fullmatch(r"mlp\.(gate|up|down)(\.b)?", rest)
        if f:
            return f"{p}.mlp.{f[1]}_proj.{'bias' if f[2] else 'weight'}"
        f = re.fullmatch(r"mix\.(left\.|right\.)?(.+)", rest)
        return f"{p}.mixer.{f[1] or ''}{self._MIX.get(f[2], f[2])}" if f else f"{p}.{rest}"

    # ---- forward ------------------------------------------------------------------------------------
    def position_tables(self, device, length: int) -> Dict[int, tuple]:
        """Per attention layer the cos / sin rows of keys and of values, one pair per two padded features (those that do not rotate
        have angle zero), for at least ``length`` positions; layers with equal constants share them."""
        out = {}
        for i, spec in enumerate(self.cfg.layer_specs):
            a = spec.attention
            if a is None:
                continue
            pair = []
            for key in ((a.rotary_dim, a.rope_theta, a.rope_factor, a.pad), (a.v_head_dim, a.rope_theta, 1.0, a.pad)):
                t = self._tables.get(key)
                if t is None or t.device != torch.device(device) or t.shape[0] < length:
                    dims, base, factor, pad = key
                    scaling = None if factor == 1.0 else {"rope_type": "linear", "factor": factor}
                    t = self._tables[key] = ops.rope_cos_sin(length, dims, base, scaling, device=device, pairs=pad // 2)
                pair.append(t)
            out[i] = tuple(pair)
        return out

    def hidden_states(self, ids, meta, kv_cache, inputs_embeds=None, capture_layers=()):
        dev = ids.device if inputs_embeds is None else inputs_embeds.device
        tables = self.position_tables(dev, meta.page_table.shape[1] * meta.page_size)
        return self.model(ids, meta, kv_cache, tables, self.comm, inputs_embeds, capture_layers)

    def logits_from_hidden(self, x: torch.Tensor, meta: StepMeta) -> torch.Tensor:
        logits = super().logits_from_hidden(x, meta)
        cap = self.cfg.final_logit_softcapping
        return ops.softcap_(logits, cap) if cap else logits

    @torch.no_grad()
    def replay_recurrent(self, record: dict, rows: torch.Tensor, meta: StepMeta, cache) -> int:
        """Besides the mixers, the input convolutions and the last token advance over the accepted rows."""
        cfg, state, m, n = self.cfg, cache.recurrent, self.model, 0
        post = lambda x, **kw: ops.stream_post(x, None, None, cfg.norm_groups, cfg.rms_norm_eps, meta, cfg.compute_dtype, **kw)
        for layer in m.layers:
            i = layer.idx
            if i not in record:
                continue
            if i == 0:
                post(None, **m.source(record["ids"].index_select(0, rows), state), **m.conv_args(0, state))
            else:
                post(record["inputs", i].index_select(0, rows), **m.conv_args(i, state))
            layer.mixer.replay(record[i], rows, meta, state, i)
            n += 1
        return n
