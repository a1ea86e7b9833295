"""Dimesun decoder: parallel layers over an fp32 residual stream, mLSTM or chunked attention beside experts, a looped span of layers.

A layer normalises once and both sublayers read that row: ``x += mult * (mixer(h) + experts(h))`` with ``h = norm(x)``.  Layers
``loop_start .. loop_stop - 1`` run ``loop_times`` times with the same weights; each run of a layer has its own cache pages or state
row, and a vector of its own is added to the stream ahead of each pass.  The stack therefore executes *runs*
(``ModelConfig.layer_run_ids``) of shared layer modules.

Per layer and step: one 16-bit product for q/k/v (and the output gate), one fp32-output product for gate pre-activations and router
logits together, the mixer, the grouped expert products, and one kernel that combines the experts, adds both sublayers to the stream,
adds the next pass's vector and normalises for the next layer (``ops.stream_norm``).
"""
from __future__ import annotations

import re
from typing import Dict, Optional

import torch
from torch import nn

from .. import ops
from ..config import LAYER_ATTENTION, LAYER_MLSTM, ModelConfig
from ..model import register_model
from ..ops.meta import StepMeta
from .default import LayerAttention
from .linear import Fp32OutLinear
from .nemotron_h import HybridCausalLM, MLstmMixer
from .qwen3_moe import GatedExperts


class OffsetRMSNorm(nn.Module):
    """RMS norm whose weight is stored around zero (gain 1 + weight); applied by ``ops.stream_norm``."""

    offset = 1.0

    def __init__(self, dim: int):
        super().__init__()
        self.weight = nn.Parameter(torch.zeros(dim, dtype=torch.float32), requires_grad=False)


class ParallelLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, idx: int):
        super().__init__()
        spec, p = cfg.layer_specs[idx], f"model.layers.{idx}"
        self.kind, self.spec = spec.kind, spec
        self.norm = OffsetRMSNorm(cfg.hidden_size)
        sizes, sources = [], []
        if spec.kind == LAYER_ATTENTION:
            self.mixer = LayerAttention(cfg, spec.attention, f"{p}.mixer")
        else:
            self.mixer = MLstmMixer(cfg, spec.mlstm, f"{p}.mixer")
            sizes += [spec.mlstm.num_heads] * 2
            sources += ["mixer.i_gate", "mixer.f_gate"]
        self.router_col = sum(sizes)
        self.mlp = None
        if spec.moe is not None:
            self.mlp = GatedExperts(cfg, spec.moe, f"{p}.mlp")
            sizes.append(spec.moe.num_experts)
            sources.append("mlp.router")
        # gate pre-activations and router logits: one product with fp32 results
        self.fp32_proj = Fp32OutLinear(cfg.hidden_size, sizes, sources=sources, bias=True, dtype=cfg.compute_dtype) if sizes else None

    def forward(self, h: torch.Tensor, meta: StepMeta, cache, cos_sin, run: int):
        """``(mixer output, expert output or None)``; the stream takes the sum."""
        small = self.fp32_proj(h) if self.fp32_proj is not None else None
        if self.kind == LAYER_ATTENTION:
            a = self.mixer(h, meta, cache.kv_layer(run), cos_sin)
        else:
            a = self.mixer(h, small, meta, cache.recurrent, run)
        if self.mlp is None:
            return a, None
        return a, self.mlp(h, small[:, self.router_col:self.router_col + self.spec.moe.num_experts])


class LoopedTransformer(nn.Module):
    def __init__(self, cfg: ModelConfig):
        super().__init__()
        self.cfg = cfg
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=cfg.compute_dtype)
        self.embed_tokens.weight.requires_grad_(False)
        self.layers = nn.ModuleList([ParallelLayer(cfg, i) for i in range(len(cfg.layer_specs))])
        self.norm = OffsetRMSNorm(cfg.hidden_size)
        self.runs = cfg.layer_run_ids
        span = cfg.loop_stop - cfg.loop_start
        if span > 0:
            self.loop_step = nn.Parameter(torch.zeros(cfg.loop_times, cfg.hidden_size, dtype=torch.float32), requires_grad=False)
            self.step_of_run: Dict[int, int] = {cfg.loop_start + t * span: t for t in range(cfg.loop_times)}
        else:
            self.loop_step, self.step_of_run = None, {}

    def _step(self, run: int) -> Optional[torch.Tensor]:
        t = self.step_of_run.get(run)
        return None if t is None else self.loop_step[t]

    def forward(self, ids, meta, cache, tables, comm, inputs_embeds=None, capture_layers=()):
        mult, eps, dt = self.cfg.residual_mult, self.cfg.rms_norm_eps, self.embed_tokens.weight.dtype
        norms = [self.layers[i].norm for i in self.runs] + [self.norm]
        table, stream = self.embed_tokens.weight, None
        if inputs_embeds is not None:
            stream = inputs_embeds.float()
        elif hasattr(table, "lookup"):                    # quantised embedding table: rows expand on lookup
            stream = ops.embedding(ids, table).float()
        x, h = ops.stream_norm(stream, norms[0].weight, eps, step=self._step(0), offset=norms[0].offset, ids=ids, table=table, dtype=dt)
        taps = []
        for run, i in enumerate(self.runs):
            layer = self.layers[i]
            a, routed = layer(h, meta, cache, tables.get(i), run)
            step = self._step(run + 1)
            if run in capture_layers:                     # the tap is the stream before the next pass's vector joins it
                x, _ = ops.stream_norm(x, None, eps, delta=a, routed=routed, mult=mult, dtype=dt)
                taps.append(x)
                a = routed = None
            x, h = ops.stream_norm(x, norms[run + 1].weight, eps, delta=a, routed=routed, mult=mult, step=step, offset=norms[run + 1].offset, dtype=dt)
        return (h, taps) if capture_layers else h


@register_model("dimesun")
class DimesunCausalLM(HybridCausalLM):
    transformer_cls = LoopedTransformer

    def __init__(self, cfg: ModelConfig, comm=None):
        if cfg.tp_size > 1 or cfg.mapping.ep_size > 1:
            raise NotImplementedError("tensor and expert parallelism are not built for the dimesun family")
        if cfg.quant.is_quantized:
            raise NotImplementedError("quantised weights are not built for the dimesun family")
        if cfg.hidden_size % 8:
            raise ValueError("the model width must be a multiple of 8")
        super().__init__(cfg, comm)
        # tied head over the embedding table, fp32 logits
        self.lm_head = Fp32OutLinear(cfg.hidden_size, [cfg.vocab_size], dtype=cfg.compute_dtype)
        self.lm_head.weight = self.model.embed_tokens.weight
        self._tables: Dict[tuple, torch.Tensor] = {}

    # ---- checkpoint names ---------------------------------------------------------------------------
    _MIX = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "g": "g_proj.weight", "o": "o_proj.weight",
            "norm": "head_norm.weight", "i": "i_gate.weight", "i.b": "i_gate.bias", "f": "f_gate.weight", "f.b": "f_gate.bias"}

    def checkpoint_key_remap(self, name: str) -> Optional[str]:
        flat = {"embed": "model.embed_tokens.weight", "loop.step": "model.loop_step", "final.norm": "model.norm.weight"}
        if name in flat:
            return flat[name]
        m = re.fullmatch(r"l(\d+)\.(.+)", name)
        if not m:
            return name
        p, rest = f"model.layers.{m[1]}", m[2]
        if rest == "norm1":
            return f"{p}.norm.weight"
        if rest.startswith("mix."):
            return f"{p}.mixer.{self._MIX.get(rest[4:], rest[4:])}"
        e = re.fullmatch(r"mlp\.e(\d+)\.(gate|up|down)", rest)
        if e:
            return f"{p}.mlp.experts.{e[1]}.{e[2]}_proj.weight"
        return {"mlp.router": f"{p}.mlp.router.weight", "mlp.router.b": f"{p}.mlp.router.bias"}.get(rest, f"{p}.{rest}")

    # ---- forward ------------------------------------------------------------------------------------
    def rope_tables(self, device, length: int) -> Dict[int, torch.Tensor]:
        """cos / sin tables per attention layer (shared by layers with the same base and size), for at least ``length`` positions."""
        out = {}
        for i, spec in enumerate(self.cfg.layer_specs):
            if spec.kind != LAYER_ATTENTION:
                continue
            a = spec.attention
            key = (a.rope_theta, a.rotary_dim)
            t = self._tables.get(key)
            if t is None or t.device != torch.device(device) or t.shape[0] < length:
                t = self._tables[key] = ops.rope_cos_sin(length, a.rotary_dim, a.rope_theta, None, device=device)
            out[i] = t
        return out

    def hidden_states(self, ids, meta, kv_cache, inputs_embeds=None, capture_layers=()):
        dev = ids.device if inputs_embeds is None else inputs_embeds.device
        tables = self.rope_tables(dev, meta.page_table.shape[1] * meta.page_size)
        return self.model(ids, meta, kv_cache, tables, self.comm, inputs_embeds, capture_layers)

    @torch.no_grad()
    def replay_recurrent(self, record: dict, rows: torch.Tensor, meta: StepMeta, cache) -> int:
        n = 0
        for run, i in enumerate(self.model.runs):
            layer = self.model.layers[i]
            if layer.kind == LAYER_MLSTM and run in record:
                layer.mixer.replay(record[run], rows, meta, cache.recurrent, run)
                n += 1
        return n
