"""Ditenex decoder: layers listed one by one over an fp32 residual stream, with a norm in front of and behind every sublayer and a token
shift before every mixer.

``h = norm1(x)``; ``h += shift * (h of the row before - h)``; ``x += mult * norm1b(mixer(h))``; ``x += mult * norm2b(mlp(norm2(x)))``.  The mixer is
windowed attention with mixed scores, the feed-forward a dense xIELU unit, or experts behind a group-limited sigmoid router beside a
shared one (or absent).  Embeddings are the sum of a token row and a position row; the head is tied to the token table.

Between two sublayers one kernel (``ops.stream_sandwich``) combines the experts, norms the sublayer's output, adds it to the stream and writes the
next norm, shifted where a mixer follows.  The last normed row of a sequence in front of each mixer is a state row indexed by seat.
"""
from __future__ import annotations

import re
from typing import Optional

import torch
from torch import nn

from .. import ops
from ..config import ModelConfig
from ..model import register_model
from ..ops.meta import StepMeta
from .default import MixedAttention, XieluMLP
from .linear import Fp32OutLinear
from .nemotron_h import HybridCausalLM
from .qwen3_moe import SharedExpertsBlock


class StreamNorm(nn.Module):
    """Weight of an RMS norm applied by ``ops.stream_sandwich``."""

    def __init__(self, dim: int):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(dim, dtype=torch.float32), requires_grad=False)


class DitenexLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, idx: int):
        super().__init__()
        spec, p, h = cfg.layer_specs[idx], f"model.layers.{idx}", cfg.hidden_size
        self.kind, self.spec, self.idx = spec.kind, spec, idx
        self.norm, self.post_norm = StreamNorm(h), StreamNorm(h)
        self.shift = nn.Parameter(torch.zeros(h, dtype=torch.float32), requires_grad=False)
        self.mixer = MixedAttention(cfg, spec.attention, f"{p}.mixer")
        self.mlp = None
        if spec.ff or spec.moe is not None:
            self.mlp_norm, self.mlp_post_norm = StreamNorm(h), StreamNorm(h)
            self.mlp = XieluMLP(cfg, spec.ff) if spec.ff else SharedExpertsBlock(cfg, spec.moe, f"{p}.mlp")

    @torch.no_grad()
    def random_init(self, gen, std=0.02):
        self.shift.copy_(torch.rand(self.shift.shape, generator=gen))

    def feed_forward(self, h: torch.Tensor):
        """``(dense rows or None, routed rows or None)``; the stream takes the sum."""
        y = self.mlp(h)
        return y if isinstance(y, tuple) else (y, None)


class DitenexTransformer(nn.Module):
    def __init__(self, cfg: ModelConfig):
        super().__init__()
        self.cfg = cfg
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=cfg.compute_dtype)
        self.embed_positions = nn.Embedding(cfg.max_position_embeddings, cfg.hidden_size, dtype=cfg.compute_dtype)
        for e in (self.embed_tokens, self.embed_positions):
            e.weight.requires_grad_(False)
        self.layers = nn.ModuleList([DitenexLayer(cfg, i) for i in range(len(cfg.layer_specs))])
        self.norm = StreamNorm(cfg.hidden_size)

    def mixer_norm(self, i: int, state) -> dict:
        """Arguments of the norm in front of mixer ``i`` (behind the last layer: the final norm)."""
        if i == len(self.layers):
            return dict(norm=self.norm.weight)
        return dict(norm=self.layers[i].norm.weight, shift=self.layers[i].shift, state=state.inputs[i])

    def forward(self, ids, meta, cache, comm, inputs_embeds=None, capture_layers=()):
        cfg, state = self.cfg, cache.recurrent
        step = lambda x, **kw: ops.stream_sandwich(x, cfg.rms_norm_eps, meta, cfg.compute_dtype, mult=cfg.residual_mult, **kw)
        rec, table, stream = state.record, self.embed_tokens.weight, None
        if inputs_embeds is not None:
            stream = inputs_embeds.float()
        elif hasattr(table, "lookup"):                    # quantised embedding table: rows expand on lookup
            stream = ops.embedding(ids, table).float()
        source = dict(ids=ids, table=table) if stream is None else {}
        x, h = step(stream, **source, positions=self.embed_positions.weight, **self.mixer_norm(0, state))
        taps, first = [], None
        for i, layer in enumerate(self.layers):
            if rec is not None:
                rec["inputs", i] = x
            y, first = layer.mixer(h, meta, cache.kv_layer(i), first)
            routed, post = None, layer.post_norm
            if layer.mlp is not None:
                x, h = step(x, delta=y, post=post.weight, norm=layer.mlp_norm.weight)
                (y, routed), post = layer.feed_forward(h), layer.mlp_post_norm
            x, h = step(x, delta=y, routed=routed, post=post.weight, **self.mixer_norm(i + 1, state))
            if i in capture_layers:
                taps.append(x)
        return (h, taps) if capture_layers else h


@register_model("ditenex")
class DitenexCausalLM(HybridCausalLM):
    transformer_cls = DitenexTransformer

    def __init__(self, cfg: ModelConfig, comm=None):
        if cfg.tp_size > 1 or cfg.mapping.ep_size > 1:
            raise NotImplementedError("tensor and expert parallelism are not built for the ditenex family")
        if cfg.quant.is_quantized:
            raise NotImplementedError("quantised weights are not built for the ditenex family")
        if cfg.hidden_size % 8:
            raise ValueError("the model width must be a multiple of 8")
        if cfg.dtype == "float16":
            raise ValueError("the ditenex family runs in bfloat16 or float32: squared activations leave the range of float16")
        super().__init__(cfg, comm)
        # tied head over the embedding table, fp32 logits
        self.lm_head = Fp32OutLinear(cfg.hidden_size, [cfg.vocab_size], dtype=cfg.compute_dtype)
        self.lm_head.weight = self.model.embed_tokens.weight

    # ---- checkpoint names ---------------------------------------------------------------------------
    _FLAT = {"embed": "model.embed_tokens.weight", "pos": "model.embed_positions.weight", "final.norm": "model.norm.weight"}
    _LAYER = {"norm1": "norm.weight", "norm1b": "post_norm.weight", "norm2": "mlp_norm.weight", "norm2b": "mlp_post_norm.weight", "shift": "shift",
              "mix.talk": "mixer.mix", "mix.vmix": "mixer.share", "mlp.act": "mlp.act", "mlp.router": "mlp.router.weight",
              "mlp.correction": "mlp.routed.correction"}

    def checkpoint_key_remap(self, name: str) -> Optional[str]:
        if name in self._FLAT:
            return self._FLAT[name]
        m = re.fullmatch(r"l(\d+)\.(.+)", name)
        if not m:
            return name
        p, rest = f"model.layers.{m[1]}", m[2]
        if rest in self._LAYER:
            return f"{p}.{self._LAYER[rest]}"
        f = re.fullmatch(r"mix\.([qkvgo])(\.b)?", rest)
        if f:
            return f"{p}.mixer.{f[1]}_proj.{'bias' if f[2] else 'weight'}"
        f = re.fullmatch(r"mlp\.(?:e(\d+)\.|(shared)\.)?(gate|up|down)", rest)
        if f:
            part = f"experts.{f[1]}." if f[1] else "shared." if f[2] else ""
            return f"{p}.mlp.{part}{f[3]}_proj.weight"
        return f"{p}.{rest}"

    # ---- forward ------------------------------------------------------------------------------------
    def hidden_states(self, ids, meta, kv_cache, inputs_embeds=None, capture_layers=()):
        return self.model(ids, meta, kv_cache, self.comm, inputs_embeds, capture_layers)

    @torch.no_grad()
    def replay_recurrent(self, record: dict, rows: torch.Tensor, meta: StepMeta, cache) -> int:
        """The last normed rows in front of the mixers advance over the accepted rows."""
        cfg, state, n = self.cfg, cache.recurrent, 0
        for i in range(len(self.model.layers)):
            x = record.get(("inputs", i))
            if x is not None:
                ops.stream_sandwich(x.index_select(0, rows), cfg.rms_norm_eps, meta, cfg.compute_dtype, **self.model.mixer_norm(i, state))
                n += 1
        return n
