"""Debonex decoder: pre-norm layers listed one by one over an fp32 residual stream, with element-wise tanh norms.

``x += mixer(norm1(x))``, then ``x += mlp(norm2(x))``; the mixer is the channel-decay delta rule, latent attention, or attention with
unit queries and keys and a query temperature; the feed-forward is a dense gated unit (or absent).  The norm keeps no statistics:
``tanh(alpha x) * weight + bias``.  Between two sublayers one kernel adds the sublayer's output to the stream and writes the next
norm (``ops.stream_norm``); the first one looks the embedding rows up and scales them.
"""
from __future__ import annotations

import re
from typing import Dict, Optional

import torch
from torch import nn

from .. import ops
from ..config import LAYER_ATTENTION, LAYER_CHANNEL_DELTA, ModelConfig
from ..model import register_model
from ..ops.meta import StepMeta
from .default import GatedMLP, LatentAttention, LayerAttention
from .linear import Fp32OutLinear
from .nemotron_h import ChannelDeltaMixer, HybridCausalLM


class TanhNorm(nn.Module):
    """``tanh(alpha x) * weight + bias``; applied by ``ops.stream_norm``."""

    def __init__(self, dim: int):
        super().__init__()
        f32 = dict(dtype=torch.float32)
        self.weight = nn.Parameter(torch.ones(dim, **f32), requires_grad=False)
        self.bias = nn.Parameter(torch.zeros(dim, **f32), requires_grad=False)
        self.alpha = nn.Parameter(torch.ones((), **f32), requires_grad=False)


class DebonexLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, idx: int):
        super().__init__()
        spec, p = cfg.layer_specs[idx], f"model.layers.{idx}"
        self.kind, self.spec, self.idx = spec.kind, spec, idx
        self.norm = TanhNorm(cfg.hidden_size)
        if spec.kind == LAYER_CHANNEL_DELTA:
            self.mixer = ChannelDeltaMixer(cfg, spec.delta, f"{p}.mixer")
        elif spec.latent is not None:
            self.mixer = LatentAttention(cfg, spec.latent, f"{p}.mixer")
        else:
            self.mixer = LayerAttention(cfg, spec.attention, f"{p}.mixer")
        if spec.ff:
            self.mlp_norm = TanhNorm(cfg.hidden_size)
            self.mlp = GatedMLP(cfg, spec.ff)
        else:
            self.mlp = None

    def mix(self, h: torch.Tensor, meta: StepMeta, cache, table) -> torch.Tensor:
        if self.kind == LAYER_ATTENTION:
            return self.mixer(h, meta, cache.kv_layer(self.idx), table)
        return self.mixer(h, meta, cache.recurrent, self.idx)


class DebonexTransformer(nn.Module):
    def __init__(self, cfg: ModelConfig):
        super().__init__()
        self.cfg = cfg
        self.embed_scale = cfg.embedding_mult
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=cfg.compute_dtype)
        self.embed_tokens.weight.requires_grad_(False)
        self.layers = nn.ModuleList([DebonexLayer(cfg, i) for i in range(len(cfg.layer_specs))])
        self.norm = TanhNorm(cfg.hidden_size)

    def forward(self, ids, meta, cache, tables, comm, inputs_embeds=None, capture_layers=()):
        eps, dt = self.cfg.rms_norm_eps, self.embed_tokens.weight.dtype
        table, source = self.embed_tokens.weight, {}
        if inputs_embeds is not None:                     # rows that already carry the embedding scale
            x = inputs_embeds.float()
        elif hasattr(table, "lookup"):                    # quantised embedding table: rows expand on lookup
            x = ops.embedding(ids, table).float() * self.embed_scale
        else:
            x, source = None, dict(ids=ids, table=table, table_mult=self.embed_scale)
        norms = [n for l in self.layers for n in ((l.norm, l.mlp_norm) if l.mlp is not None else (l.norm,))] + [self.norm]
        advance = lambda x, delta, n, **kw: ops.stream_norm(x, n.weight, eps, delta=delta, alpha=n.alpha, bias=n.bias, dtype=dt, **kw)
        x, h = advance(x, None, norms[0], **source)
        taps, at = [], 1
        for i, layer in enumerate(self.layers):
            x, h = advance(x, layer.mix(h, meta, cache, tables.get(i)), norms[at])
            at += 1
            if layer.mlp is not None:
                x, h = advance(x, layer.mlp(h), norms[at])
                at += 1
            if i in capture_layers:
                taps.append(x)
        return (h, taps) if capture_layers else h


@register_model("debonex")
class DebonexCausalLM(HybridCausalLM):
    transformer_cls = DebonexTransformer

    def __init__(self, cfg: ModelConfig, comm=None):
        if cfg.tp_size > 1 or cfg.mapping.ep_size > 1:
            raise NotImplementedError("tensor and expert parallelism are not built for the debonex family")
        if cfg.quant.is_quantized:
            raise NotImplementedError("quantised weights are not built for the debonex family")
        if cfg.hidden_size % 8:
            raise ValueError("the model width must be a multiple of 8")
        super().__init__(cfg, comm)
        self.lm_head = Fp32OutLinear(cfg.hidden_size, [cfg.vocab_size], dtype=cfg.compute_dtype)
        self._tables: Dict[tuple, torch.Tensor] = {}

    # ---- checkpoint names ---------------------------------------------------------------------------
    _MIX = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "o": "o_proj.weight", "b": "beta_proj.weight",
            "q.conv": "q_conv", "k.conv": "k_conv", "v.conv": "v_conv", "a1": "decay_in_proj.weight", "a2": "decay_out_proj.weight",
            "g1": "gate_in_proj.weight", "g2": "gate_out_proj.weight", "A_log": "a_log", "norm": "head_norm.weight",
            "dkv": "kv_down_proj.weight", "dkv.norm": "latent_norm.weight", "uk": "k_up_proj.weight", "uv": "v_up_proj.weight"}
    _NORM = {"": "weight", ".b": "bias", ".alpha": "alpha"}

    def checkpoint_key_remap(self, name: str) -> Optional[str]:
        flat = {"embed": "model.embed_tokens.weight", "head": "lm_head.weight"}
        if name in flat:
            return flat[name]
        m = re.fullmatch(r"(?:final|l(\d+))\.norm([12]?)(|\.b|\.alpha)", name)
        if m:
            layer = "model.norm" if m[1] is None else f"model.layers.{m[1]}.{'mlp_norm' if m[2] == '2' else 'norm'}"
            return f"{layer}.{self._NORM[m[3]]}"
        m = re.fullmatch(r"l(\d+)\.(mix|mlp)\.(.+)", name)
        if not m:
            return name
        p = f"model.layers.{m[1]}"
        return f"{p}.mixer.{self._MIX.get(m[3], m[3])}" if m[2] == "mix" else f"{p}.mlp.{m[3]}_proj.weight"

    # ---- forward ------------------------------------------------------------------------------------
    def position_tables(self, device, length: int) -> Dict[int, torch.Tensor]:
        """Per layer with positions: cos / sin rows of latent attention, or query temperatures (layers with equal constants share
        one); for at least ``length`` positions."""
        out = {}
        for i, spec in enumerate(self.cfg.layer_specs):
            if spec.latent is not None:
                key, make = ("rot", spec.latent.rope_theta, spec.latent.rot_dim), lambda n, k: ops.rope_cos_sin(n, k[2], k[1], None, device=device)
            elif spec.attention is not None:
                key, make = ("temp", spec.attention.temp_coef, spec.attention.temp_every), lambda n, k: ops.query_temperature(n, k[1], k[2], device)
            else:
                continue
            t = self._tables.get(key)
            if t is None or t.device != torch.device(device) or t.shape[0] < length:
                t = self._tables[key] = make(length, key)
            out[i] = t
        return out

    def hidden_states(self, ids, meta, kv_cache, inputs_embeds=None, capture_layers=()):
        dev = ids.device if inputs_embeds is None else inputs_embeds.device
        tables = self.position_tables(dev, meta.page_table.shape[1] * meta.page_size)
        return self.model(ids, meta, kv_cache, tables, self.comm, inputs_embeds, capture_layers)

    def logits_from_hidden(self, x: torch.Tensor, meta: StepMeta) -> torch.Tensor:
        logits = super().logits_from_hidden(x, meta)
        return logits if self.cfg.logits_mult == 1.0 else logits.mul_(self.cfg.logits_mult)

    @torch.no_grad()
    def replay_recurrent(self, record: dict, rows: torch.Tensor, meta: StepMeta, cache) -> int:
        n = 0
        for layer in self.model.layers:
            if layer.kind == LAYER_CHANNEL_DELTA and layer.idx in record:
                layer.mixer.replay(record[layer.idx], rows, meta, cache.recurrent, layer.idx)
                n += 1
        return n
