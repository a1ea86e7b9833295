"""Hybrid decoder: Mamba2-SSD, gated-DeltaNet and GQA-attention mixers with dense MLPs.

Parity: ``tensorrt_edgellm/models/nemotron_h/modeling_nemotron_h.py`` — ``MambaMixer`` wiring
(:239-446: ``in_proj → [z | conv-in (x‖B‖C) | dt]``, conv1d + SiLU, ``A = −exp(A_log)``, selective
state update, gated group-RMSNorm, ``out_proj``; dt clamp), relu² MLP (:555-573) — and the gated
DeltaNet mixer of ``tensorrt_edgellm/models/qwen3_5/modeling_qwen3_5_text.py:162-379`` (``in_proj_qkv
‖ z ‖ b ‖ a``, conv1d + SiLU, delta rule, per-head RMSNorm · silu(z), ``out_proj``).

A layer is ``x += mixer(norm(x))`` followed by ``x += mlp(norm(x))``; either half may be absent
(``layer_types[i] == "none"`` / ``mlp_types[i] == "none"``), which covers both the Nemotron-H
block pattern (one mixer *or* one MLP per block) and transformer-style hybrid stacks.  Recurrent
state (conv history, SSM state, delta-rule state) lives in per-layer pools indexed by the step's
``slot_ids``; tensor parallelism shards heads (column-parallel in, row-parallel out).
"""
from __future__ import annotations

from typing import Optional

import torch
from torch import nn

from .. import ops
from ..config import (LAYER_ATTENTION, LAYER_CHANNEL_DELTA, LAYER_GDN, LAYER_LIGHTNING, LAYER_MAMBA, LAYER_MLP, LAYER_MLSTM, LAYER_MOE, LAYER_PARALLEL,
                      ModelConfig)
from ..model import register_model
from ..ops.meta import StepMeta
from .default import MLP, Attention, CausalLM, LayerAttention, RMSNorm
from .linear import Fp32OutLinear, HeadLinear, JoinedLinear, StackedRankLinear, TPMode, make_linear


class RecurrentState:
    """Per-layer state pools of the recurrent mixers (rows = seats)."""

    def __init__(self, cfg: ModelConfig, seats: int, device, dtype):
        tp = cfg.tp_size
        self.conv, self.ssm, self.gdn = {}, {}, {}
        self.mlstm, self.mlstm_norm = {}, {}      # matrix memory; normaliser and running maximum
        self.delta = {}                           # delta rule with a decay per key channel or head
        self.lightning = {}                       # linear attention with constant decays
        self.inputs = {}                          # last rows in front of each mixer (of the stream: input convolution; normed: token shift), fp32
        self.tokens = {}                          # the sequence's last token (bigram embeddings)
        runs = cfg.layer_run_ids if cfg.layer_specs else None
        for i, t in enumerate(cfg.layer_types):
            if t == LAYER_MAMBA:
                m = cfg.mamba
                conv_dim = (m.intermediate_size + 2 * m.n_groups * m.d_state) // tp
                self.conv[i] = torch.zeros(seats, conv_dim, m.conv_kernel - 1, dtype=dtype, device=device)
                self.ssm[i] = torch.zeros(seats, m.num_heads // tp, m.head_dim, m.d_state, dtype=torch.float32, device=device)
            elif t == LAYER_GDN:
                g = cfg.gdn
                self.conv[i] = torch.zeros(seats, g.conv_dim // tp, g.conv_kernel - 1, dtype=dtype, device=device)
                self.gdn[i] = torch.zeros(seats, g.num_v_heads // tp, g.head_k_dim, g.head_v_dim, dtype=torch.float32, device=device)

            elif t == LAYER_MLSTM:
                m = cfg.layer_specs[runs[i]].mlstm
                self.mlstm[i] = torch.zeros(seats, m.num_heads, m.k_pad, m.v_pad, dtype=torch.float32, device=device)
                self.mlstm_norm[i] = torch.zeros(seats, m.num_heads, m.k_pad + 1, dtype=torch.float32, device=device)
            elif t in (LAYER_CHANNEL_DELTA, LAYER_PARALLEL):
                d = cfg.layer_specs[runs[i]].delta
                self.conv[i] = torch.zeros(seats, d.conv_dim, d.conv_kernel - 1, dtype=dtype, device=device)
                self.delta[i] = torch.zeros(seats, d.num_heads, d.k_pad, d.v_pad, dtype=torch.float32, device=device)
            elif t == LAYER_LIGHTNING:
                l = cfg.layer_specs[runs[i]].lightning
                self.lightning[i] = torch.zeros(seats, l.num_heads, l.k_pad, l.v_pad, dtype=torch.float32, device=device)
            if cfg.input_conv > 1 or cfg.token_shift:
                rows = 1 if cfg.token_shift else cfg.input_conv - 1
                self.inputs[i] = torch.zeros(seats, rows, cfg.hidden_size, dtype=torch.float32, device=device)
        if cfg.bigram_buckets:
            self.tokens[0] = torch.zeros(seats, 1, dtype=torch.int32, device=device)

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.pools())

    def pools(self):
        for d in (self.conv, self.ssm, self.gdn, self.mlstm, self.mlstm_norm, self.delta, self.lightning, self.inputs, self.tokens):
            yield from d.values()

    # ---- replay data -------------------------------------------------------------------------------------------------
    # A speculative verification step advances every state over the whole draft chain.  While ``record`` is a dict the mixers
    # also keep the inputs of their recurrent kernels for that step (a few KB per token and layer); when only a prefix of
    # the chain is accepted, ``HybridCausalLM.replay_recurrent`` restores the saved rows and runs *only the recurrent kernels*
    # over the accepted tokens again from those inputs: no projections, no attention, no MLP.
    record = None

    def begin_record(self) -> None:
        self.record = {}

    def end_record(self):
        rec, self.record = self.record, None
        return rec

    def snapshot(self, seats) -> list:
        """Copies of the state rows of ``seats`` (the commit policy of speculative verification restores them when a
        draft chain is only partly accepted; ``cpp/runtime/commitPolicy/`` in the reference)."""
        idx = torch.as_tensor(list(seats), dtype=torch.long, device=next(self.pools()).device)
        return [t.index_select(0, idx) for t in self.pools()]

    def restore(self, seats, snap: list, which=None) -> None:
        """Write back the rows of ``snap`` for ``seats`` (all of them, or the positions listed in ``which``)."""
        sel = list(range(len(seats))) if which is None else list(which)
        if not sel:
            return
        dev = next(self.pools()).device
        dst = torch.as_tensor([seats[j] for j in sel], dtype=torch.long, device=dev)
        src = torch.as_tensor(sel, dtype=torch.long, device=dev)
        for t, saved in zip(self.pools(), snap):
            t.index_copy_(0, dst, saved.index_select(0, src))


class MambaMixer(nn.Module):
    def __init__(self, cfg: ModelConfig, prefix: str):
        super().__init__()
        m, tp = cfg.mamba, cfg.tp_size
        self.m = m
        self.nheads = m.num_heads // tp
        self.groups = max(m.n_groups // tp, 1)
        if m.num_heads % tp or m.n_groups % tp:
            raise ValueError("Mamba heads and groups must divide over the TP ranks")
        self.d_inner = self.nheads * m.head_dim
        self.bc = self.groups * m.d_state
        di, gn = m.intermediate_size, m.n_groups * m.d_state
        # one checkpoint tensor in_proj.weight = [z | x | B | C | dt]; each segment is sharded on its own
        self.in_proj = make_linear(cfg, f"{prefix}.in_proj", cfg.hidden_size, [di, di, gn, gn, m.num_heads], TPMode.COL)
        self.out_proj = make_linear(cfg, f"{prefix}.out_proj", di, [cfg.hidden_size], TPMode.ROW)
        conv_dim = self.d_inner + 2 * self.bc
        dt = cfg.compute_dtype
        self.conv_weight = nn.Parameter(torch.zeros(conv_dim, m.conv_kernel, dtype=dt), requires_grad=False)
        self.conv_bias = nn.Parameter(torch.zeros(conv_dim, dtype=dt), requires_grad=False)
        self.A_log = nn.Parameter(torch.zeros(self.nheads, dtype=torch.float32), requires_grad=False)
        self.D = nn.Parameter(torch.ones(self.nheads, dtype=torch.float32), requires_grad=False)
        self.dt_bias = nn.Parameter(torch.zeros(self.nheads, dtype=torch.float32), requires_grad=False)
        self.norm_weight = nn.Parameter(torch.ones(self.d_inner, dtype=dt), requires_grad=False)
        self.eps = cfg.rms_norm_eps
        self.prefix, self.cfg = prefix, cfg

    @torch.no_grad()
    def load_checkpoint(self, fetch) -> bool:
        w = fetch(f"{self.prefix}.conv1d.weight")
        if w is None:
            return False
        m, tp, r = self.m, self.cfg.tp_size, self.cfg.tp_rank
        di, gn = m.intermediate_size, m.n_groups * m.d_state

        def seg(t):     # shard [x | B | C] stacked along dim 0
            parts = [t[:di], t[di:di + gn], t[di + gn:di + 2 * gn]]
            return torch.cat([p.chunk(tp, 0)[r] for p in parts], 0)

        self.conv_weight.copy_(seg(w.reshape(w.shape[0], -1)).to(self.conv_weight.dtype))
        b = fetch(f"{self.prefix}.conv1d.bias")
        if b is not None:
            self.conv_bias.copy_(seg(b).to(self.conv_bias.dtype))
        for name, dst in (("A_log", self.A_log), ("D", self.D), ("dt_bias", self.dt_bias)):
            t = fetch(f"{self.prefix}.{name}")
            if t is not None:
                dst.copy_(t.float().chunk(tp, 0)[r])
        nw = fetch(f"{self.prefix}.norm.weight")
        if nw is not None:
            self.norm_weight.copy_(nw.chunk(tp, 0)[r].to(self.norm_weight.dtype))
        return False        # linear layers are still loaded by the generic path

    @torch.no_grad()
    def random_init(self, gen, std=0.02):
        self.conv_weight.copy_((torch.randn(self.conv_weight.shape, generator=gen) * 0.3).to(self.conv_weight.dtype))
        self.A_log.copy_(torch.log(torch.rand(self.nheads, generator=gen) * 3 + 1))
        self.dt_bias.copy_(torch.rand(self.nheads, generator=gen) - 2.0)

    def forward(self, x, meta: StepMeta, state: RecurrentState, layer_idx: int):
        m = self.m
        proj = self.in_proj(x)
        z, xbc, dt = proj.split([self.d_inner, self.d_inner + 2 * self.bc, self.nheads], dim=-1)
        if state.record is not None:
            state.record[layer_idx] = (xbc.contiguous(), dt.contiguous())
        xbc = ops.causal_conv1d(xbc.contiguous(), self.conv_weight, self.conv_bias, state.conv[layer_idx], meta, activation=True)
        xs, B, C = xbc.split([self.d_inner, self.bc, self.bc], dim=-1)
        t = x.shape[0]
        y = ops.ssm_scan(xs.reshape(t, self.nheads, m.head_dim), dt.contiguous(), -torch.exp(self.A_log),
                         B.reshape(t, self.groups, m.d_state), C.reshape(t, self.groups, m.d_state), self.D, self.dt_bias,
                         state.ssm[layer_idx], meta, z=None, dt_softplus=True, dt_limit=m.dt_limit)
        y = ops.gated_group_rmsnorm(y.reshape(t, self.d_inner), z.contiguous(), self.norm_weight, self.groups, self.eps)
        return self.out_proj(y)


    @torch.no_grad()
    def replay(self, saved, rows: torch.Tensor, meta: StepMeta, state: RecurrentState, layer_idx: int) -> None:
        """Advance this layer's convolution and SSM state over the recorded inputs of ``rows`` (the accepted tokens)."""
        m = self.m
        xbc, dt = (t.index_select(0, rows) for t in saved)
        xbc = ops.causal_conv1d(xbc, self.conv_weight, self.conv_bias, state.conv[layer_idx], meta, activation=True)
        xs, B, C = xbc.split([self.d_inner, self.bc, self.bc], dim=-1)
        t = xbc.shape[0]
        ops.ssm_scan(xs.reshape(t, self.nheads, m.head_dim), dt, -torch.exp(self.A_log), B.reshape(t, self.groups, m.d_state),
                     C.reshape(t, self.groups, m.d_state), self.D, self.dt_bias, state.ssm[layer_idx], meta, z=None, dt_softplus=True,
                     dt_limit=m.dt_limit)


class GatedDeltaNetMixer(nn.Module):
    def __init__(self, cfg: ModelConfig, prefix: str):
        super().__init__()
        g, tp = cfg.gdn, cfg.tp_size
        self.g = g
        if g.num_k_heads % tp or g.num_v_heads % tp:
            raise ValueError("gated-DeltaNet heads must divide over the TP ranks")
        self.hk, self.hv = g.num_k_heads // tp, g.num_v_heads // tp
        self.key_dim, self.value_dim = self.hk * g.head_k_dim, self.hv * g.head_v_dim
        h = cfg.hidden_size
        self.in_proj_qkv = make_linear(cfg, f"{prefix}.in_proj_qkv", h, [g.key_dim, g.key_dim, g.value_dim], TPMode.COL)
        self.in_proj_z = make_linear(cfg, f"{prefix}.in_proj_z", h, [g.value_dim], TPMode.COL)
        self.in_proj_b = make_linear(cfg, f"{prefix}.in_proj_b", h, [g.num_v_heads], TPMode.COL, quantizable=False)
        self.in_proj_a = make_linear(cfg, f"{prefix}.in_proj_a", h, [g.num_v_heads], TPMode.COL, quantizable=False)
        self.out_proj = make_linear(cfg, f"{prefix}.out_proj", g.value_dim, [h], TPMode.ROW)
        dt = cfg.compute_dtype
        conv_dim = 2 * self.key_dim + self.value_dim
        self.conv_weight = nn.Parameter(torch.zeros(conv_dim, g.conv_kernel, dtype=dt), requires_grad=False)
        self.A_log = nn.Parameter(torch.zeros(self.hv, dtype=torch.float32), requires_grad=False)
        self.dt_bias = nn.Parameter(torch.zeros(self.hv, dtype=torch.float32), requires_grad=False)
        self.norm_weight = nn.Parameter(torch.ones(g.head_v_dim, dtype=dt), requires_grad=False)
        self.eps = cfg.rms_norm_eps
        self.prefix, self.cfg = prefix, cfg

    @torch.no_grad()
    def load_checkpoint(self, fetch) -> bool:
        w = fetch(f"{self.prefix}.conv1d.weight")
        if w is None:
            return False
        g, tp, r = self.g, self.cfg.tp_size, self.cfg.tp_rank
        w = w.reshape(w.shape[0], -1)
        parts = [w[:g.key_dim], w[g.key_dim:2 * g.key_dim], w[2 * g.key_dim:]]
        self.conv_weight.copy_(torch.cat([p.chunk(tp, 0)[r] for p in parts], 0).to(self.conv_weight.dtype))
        for name, dst in (("A_log", self.A_log), ("dt_bias", self.dt_bias)):
            t = fetch(f"{self.prefix}.{name}")
            if t is not None:
                dst.copy_(t.float().chunk(tp, 0)[r])
        nw = fetch(f"{self.prefix}.norm.weight")
        if nw is not None:
            self.norm_weight.copy_(nw.to(self.norm_weight.dtype))
        return False

    @torch.no_grad()
    def random_init(self, gen, std=0.02):
        self.conv_weight.copy_((torch.randn(self.conv_weight.shape, generator=gen) * 0.3).to(self.conv_weight.dtype))
        self.A_log.copy_(torch.log(torch.rand(self.hv, generator=gen) * 3 + 1))
        self.dt_bias.copy_(torch.rand(self.hv, generator=gen) - 2.0)

    def forward(self, x, meta: StepMeta, state: RecurrentState, layer_idx: int):
        g = self.g
        t = x.shape[0]
        qkv = self.in_proj_qkv(x)
        z = self.in_proj_z(x)
        b = self.in_proj_b(x)
        a = self.in_proj_a(x)
        if state.record is not None:
            state.record[layer_idx] = (qkv.contiguous(), a.contiguous(), b.contiguous())
        qkv = ops.causal_conv1d(qkv, self.conv_weight, None, state.conv[layer_idx], meta, activation=True)
        q, k, v = qkv.split([self.key_dim, self.key_dim, self.value_dim], dim=-1)
        o = ops.gated_delta_rule(q.reshape(t, self.hk, g.head_k_dim), k.reshape(t, self.hk, g.head_k_dim),
                                 v.reshape(t, self.hv, g.head_v_dim), a, b, self.A_log, self.dt_bias, state.gdn[layer_idx], meta)
        # per-head RMSNorm, then the silu(z) gate
        o = ops.rmsnorm(o.reshape(t * self.hv, g.head_v_dim).contiguous(), self.norm_weight, self.eps).reshape(t, self.value_dim)
        zf = z.float()
        o = (o.float() * (zf * torch.sigmoid(zf))).to(x.dtype)
        return self.out_proj(o)


    @torch.no_grad()
    def replay(self, saved, rows: torch.Tensor, meta: StepMeta, state: RecurrentState, layer_idx: int) -> None:
        g = self.g
        qkv, a, b = (t.index_select(0, rows) for t in saved)
        qkv = ops.causal_conv1d(qkv, self.conv_weight, None, state.conv[layer_idx], meta, activation=True)
        q, k, v = qkv.split([self.key_dim, self.key_dim, self.value_dim], dim=-1)
        t = qkv.shape[0]
        ops.gated_delta_rule(q.reshape(t, self.hk, g.head_k_dim), k.reshape(t, self.hk, g.head_k_dim), v.reshape(t, self.hv, g.head_v_dim),
                             a, b, self.A_log, self.dt_bias, state.gdn[layer_idx], meta)


class MLstmMixer(nn.Module):
    """Matrix-memory LSTM: q, k, v and the output gate from one product; the log input and forget gates arrive as fp32 columns of the
    layer's fp32 projection (``gates``: input gates of all heads, then forget gates); state in fp32 rows indexed by seat.  Head norm
    and output gate are part of the recurrent op."""

    def __init__(self, cfg: ModelConfig, spec, prefix: str):
        super().__init__()
        self.spec, self.prefix, self.eps = spec, prefix, cfg.rms_norm_eps
        h, n, dt = cfg.hidden_size, spec.num_heads, cfg.compute_dtype
        self.qkvg_proj = HeadLinear(h, 0, out_heads=[(n, spec.head_k_dim, spec.k_pad), (n, spec.head_k_dim, spec.k_pad),
                                                     (n, spec.head_v_dim, spec.v_pad), (n, spec.head_v_dim, spec.v_pad)],
                                    sources=["q_proj", "k_proj", "v_proj", "g_proj"], dtype=dt)
        self.o_proj = HeadLinear(0, h, in_heads=(n, spec.head_v_dim, spec.v_pad), dtype=dt)
        self.out_norm = nn.Parameter(torch.ones(n * spec.v_pad, dtype=torch.float32), requires_grad=False)

    @torch.no_grad()
    def load_checkpoint(self, fetch) -> bool:
        w = fetch(f"{self.prefix}.head_norm.weight")
        if w is not None:
            sp = self.spec
            self.out_norm.zero_()
            self.out_norm.view(sp.num_heads, sp.v_pad)[:, :sp.head_v_dim] = w.float().reshape(sp.num_heads, sp.head_v_dim)
        return False        # the projections are loaded by the generic path

    def forward(self, x, gates, meta: StepMeta, state: RecurrentState, run: int):
        qkvg = self.qkvg_proj(x)
        if state.record is not None:
            state.record[run] = (qkvg, gates)
        return self.o_proj(self._recur(qkvg, gates, meta, state, run))

    def _recur(self, qkvg, gates, meta, state, run):
        sp = self.spec
        return ops.mlstm(qkvg, gates, self.out_norm, state.mlstm[run], state.mlstm_norm[run], meta, sp.head_k_dim ** -0.5, sp.gate_cap,
                         self.eps, sp.head_v_dim)

    @torch.no_grad()
    def replay(self, saved, rows: torch.Tensor, meta: StepMeta, state: RecurrentState, run: int) -> None:
        self._recur(*(t.index_select(0, rows) for t in saved), meta, state, run)


class ChannelDeltaMixer(nn.Module):
    """Delta rule with one decay per head and key channel, or (``head_decay``) one per head.

    Per channel: q, k and v come from one product; the inner rows of the two low-rank projections (decays, output gate) from a second,
    their outer halves and the step sizes with fp32 results.  Per head: q, k, v and the gate from one product, step sizes and decays from a
    second with fp32 results.  Short convolutions, unit norms, decays, recurrence, head norm and output gate are one op over the
    step's rows (``ops.channel_delta``).  ``bare``: no projections; a surrounding mixer hands the rows to :meth:`recur`."""

    def __init__(self, cfg: ModelConfig, spec, prefix: str, bare: bool = False):
        super().__init__()
        self.spec, self.prefix, self.eps = spec, prefix, cfg.rms_norm_eps
        h, n, nk, dt = cfg.hidden_size, spec.num_heads, spec.num_kv_heads, cfg.compute_dtype
        self.row_heads = [(nk, spec.head_k_dim, spec.k_pad), (nk, spec.head_k_dim, spec.k_pad), (n, spec.head_v_dim, spec.v_pad)]
        self.out_heads = (n, spec.head_v_dim, spec.v_pad)
        if bare:
            pass
        elif spec.head_decay:
            self.qkvg_proj = HeadLinear(h, 0, out_heads=self.row_heads + [self.out_heads], sources=["q_proj", "k_proj", "v_proj", "g_proj"], dtype=dt)
            self.beta_decay_proj = Fp32OutLinear(h, [n, n], sources=["beta_proj", "decay_proj"], dtype=dt)
        else:
            self.qkv_proj = HeadLinear(h, 0, out_heads=self.row_heads, sources=["q_proj", "k_proj", "v_proj"], dtype=dt)
            ranks = [(1, r, (r + 7) // 8 * 8) for r in (spec.decay_rank, spec.gate_rank)]
            self.rank_proj = HeadLinear(h, 0, out_heads=ranks, sources=["decay_in_proj", "gate_in_proj"], dtype=dt)
            self.up_proj = StackedRankLinear(ranks, [(n, spec.head_k_dim, spec.k_pad), self.out_heads],
                                             sources=["decay_out_proj", "gate_out_proj"], dtype=dt)
            self.beta_proj = Fp32OutLinear(h, [n], dtype=dt)
        if not bare:
            self.o_proj = HeadLinear(0, h, in_heads=self.out_heads, dtype=dt)
        self.conv_weight = nn.Parameter(torch.zeros(spec.conv_dim, spec.conv_kernel, dtype=dt), requires_grad=False)
        self.a_log = nn.Parameter(torch.zeros(n, dtype=torch.float32), requires_grad=False)
        self.decay_bias = nn.Parameter(torch.zeros(n if spec.head_decay else n * spec.k_pad, dtype=torch.float32), requires_grad=False)
        self.norm_weight = nn.Parameter(torch.ones(spec.v_pad, dtype=torch.float32), requires_grad=False)

    def _heads(self, t: torch.Tensor, heads: int, real: int, pad: int) -> torch.Tensor:
        """``[heads * real, ...]`` checkpoint rows with every head padded by zero rows."""
        t = t.reshape(heads, real, -1)
        return torch.nn.functional.pad(t, (0, 0, 0, pad - real)).reshape(heads * pad, -1)

    @torch.no_grad()
    def load_checkpoint(self, fetch) -> bool:
        sp = self.spec
        taps = [fetch(f"{self.prefix}.{n}_conv") for n in "qkv"]
        if any(t is None for t in taps):
            return False
        self.conv_weight.copy_(torch.cat([self._heads(t, *z) for t, z in zip(taps, self.row_heads)]).to(self.conv_weight.dtype))
        bias = fetch(f"{self.prefix}.dt_bias").float()
        self.decay_bias.copy_(bias if sp.head_decay else self._heads(bias, sp.num_heads, sp.head_k_dim, sp.k_pad)[:, 0])
        self.norm_weight.zero_()
        self.norm_weight[:sp.head_v_dim] = fetch(f"{self.prefix}.head_norm.weight").float()
        return False        # the projections and a_log are loaded by the generic path

    @torch.no_grad()
    def random_init(self, gen, std=0.02):
        self.conv_weight.copy_((torch.randn(self.conv_weight.shape, generator=gen) * 0.3).to(self.conv_weight.dtype))
        self.a_log.copy_(torch.rand(self.spec.num_heads, generator=gen))
        self.decay_bias.copy_(torch.rand(self.decay_bias.shape, generator=gen) - 4.0)

    def forward(self, x, meta: StepMeta, state: RecurrentState, run: int):
        n, sp = self.spec.num_heads, self.spec
        if sp.head_decay:
            rows, small = self.qkvg_proj(x), self.beta_decay_proj(x)
            saved = (rows[:, :sp.conv_dim], small[:, n:], rows[:, sp.conv_dim:], small[:, :n])
        else:
            qkv, beta = self.qkv_proj(x), self.beta_proj(x)
            decay, gate = self.up_proj(self.rank_proj(x))
            saved = (qkv, decay, gate, beta)
        if state.record is not None:
            state.record[run] = saved
        return self.o_proj(self.recur(*saved, meta, state, run))

    def recur(self, qkv, decay, gate, beta, meta, state, run, out: Optional[torch.Tensor] = None, mult: float = 1.0):
        """Gated head outputs of packed rows and pre-activations (into ``out``, times ``mult``)."""
        return ops.channel_delta(qkv, decay, gate, beta, self.conv_weight, self.a_log, self.decay_bias, self.norm_weight, state.conv[run],
                                 state.delta[run], meta, self.spec, self.eps, out=out, mult=mult)

    @torch.no_grad()
    def replay(self, saved, rows: torch.Tensor, meta: StepMeta, state: RecurrentState, run: int) -> None:
        self.recur(*(t.index_select(0, rows) for t in saved), meta, state, run)


class LightningMixer(nn.Module):
    """Linear attention with a constant decay per head: q, k, v and the output gate from one product; silu, recurrence, norm weight and
    gate are one op (``ops.lightning``); state in fp32 rows indexed by seat.  The root mean square over all heads of a row commutes with
    the output projection: ``forward`` returns the projected rows and the sums that their consumer divides by."""

    POWERS = 256          # decay^0 .. decay^POWERS, rounded once from double

    def __init__(self, cfg: ModelConfig, spec, prefix: str):
        super().__init__()
        self.spec, self.prefix = spec, prefix
        h, n, dt = cfg.hidden_size, spec.num_heads, cfg.compute_dtype
        self.qkvg_proj = HeadLinear(h, 0, out_heads=[(n, spec.head_k_dim, spec.k_pad), (n, spec.head_k_dim, spec.k_pad),
                                                     (n, spec.head_v_dim, spec.v_pad), (n, spec.head_v_dim, spec.v_pad)],
                                    sources=["q_proj", "k_proj", "v_proj", "g_proj"], dtype=dt)
        self.o_proj = HeadLinear(0, h, in_heads=(n, spec.head_v_dim, spec.v_pad), dtype=dt)
        self.out_norm = nn.Parameter(torch.ones(n * spec.v_pad, dtype=torch.float32), requires_grad=False)
        decay = torch.tensor([float(x) for x in spec.decay], dtype=torch.float64)[:, None]
        steps = torch.arange(self.POWERS + 1, dtype=torch.float64, device=decay.device)
        self.register_buffer("decay_powers", (decay ** steps).float(), persistent=False)

    @torch.no_grad()
    def load_checkpoint(self, fetch) -> bool:
        w = fetch(f"{self.prefix}.head_norm.weight")
        if w is not None:
            sp = self.spec
            self.out_norm.zero_()
            self.out_norm.view(sp.num_heads, sp.v_pad)[:, :sp.head_v_dim] = w.float().reshape(sp.num_heads, sp.head_v_dim)
        return False        # the projections are loaded by the generic path

    def forward(self, x, meta: StepMeta, state: RecurrentState, run: int):
        rows = self.qkvg_proj(x)
        if state.record is not None:
            state.record[run] = rows
        u, sums = self._recur(rows, meta, state, run)
        return self.o_proj(u), (sums, self.spec.num_heads * self.spec.head_v_dim)

    def _recur(self, rows, meta, state, run):
        return ops.lightning(rows, self.out_norm, self.decay_powers, state.lightning[run], meta)

    @torch.no_grad()
    def replay(self, saved, rows: torch.Tensor, meta: StepMeta, state: RecurrentState, run: int) -> None:
        self._recur(saved.index_select(0, rows), meta, state, run)


class ParallelMixer(nn.Module):
    """Attention and a delta rule on the same input, ``attention_mult * attention + delta_mult * delta``.  One product gives the rows of both,
    a small one with fp32 results the step sizes and decays; both write their heads into one row, and one product over it is the
    weighted sum of the two output projections (the multipliers join the heads in fp32)."""

    def __init__(self, cfg: ModelConfig, spec, prefix: str):
        super().__init__()
        self.spec, h, dt = spec, cfg.hidden_size, cfg.compute_dtype
        self.left = LayerAttention(cfg, spec.attention, f"{prefix}.left", bare=True)
        self.right = ChannelDeltaMixer(cfg, spec.delta, f"{prefix}.right", bare=True)
        heads = self.left.row_heads + self.right.row_heads + [self.right.out_heads]
        self.in_proj = HeadLinear(h, 0, out_heads=heads, dtype=dt, sources=[f"left.{n}_proj" for n in "qkv"] + [f"right.{n}_proj" for n in "qkvg"])
        n = spec.delta.num_heads
        self.beta_decay_proj = Fp32OutLinear(h, [n, n], sources=["right.beta_proj", "right.decay_proj"], dtype=dt)
        self.out_proj = JoinedLinear([self.left.out_heads, self.right.out_heads], h, sources=["left.o_proj", "right.o_proj"], dtype=dt)
        width = lambda heads: sum(h * pad for h, _, pad in heads)
        self.left_cols, self.right_cols = width(self.left.row_heads), width(self.right.row_heads)
        self.left_out = width([self.left.out_heads])

    def forward(self, x, meta: StepMeta, cache, table, run: int):
        rows, small, state = self.in_proj(x), self.beta_decay_proj(x), cache.recurrent
        n, c = self.spec.delta.num_heads, self.left_cols + self.right_cols
        delta_in = (rows[:, self.left_cols:c], small[:, n:], rows[:, c:], small[:, :n])
        if state.record is not None:
            state.record[run] = delta_in
        y = torch.empty(x.shape[0], self.out_proj.in_features, dtype=x.dtype, device=x.device)
        self.left.attend(rows[:, :self.left_cols], meta, cache.kv_layer(run), table, out=y[:, :self.left_out], mult=self.spec.attention_mult)
        self.right.recur(*delta_in, meta, state, run, out=y[:, self.left_out:], mult=self.spec.delta_mult)
        return self.out_proj(y)

    @torch.no_grad()
    def replay(self, saved, rows: torch.Tensor, meta: StepMeta, state: RecurrentState, run: int) -> None:
        self.right.replay(saved, rows, meta, state, run)


class HybridLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, i: int):
        super().__init__()
        p = f"model.layers.{i}"
        kind, mlp_kind = cfg.layer_types[i], cfg.mlp_types[i]
        self.kind, self.mlp_kind, self.idx = kind, mlp_kind, i
        dt = cfg.compute_dtype
        if kind == LAYER_ATTENTION:
            self.mixer = Attention(cfg, i, f"{p}.mixer")
        elif kind == LAYER_MAMBA:
            self.mixer = MambaMixer(cfg, f"{p}.mixer")
        elif kind == LAYER_GDN:
            self.mixer = GatedDeltaNetMixer(cfg, f"{p}.mixer")
        else:
            self.mixer = None
        if self.mixer is not None:
            self.norm = RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, dt)
        if mlp_kind == LAYER_MLP:
            self.mlp = MLP(cfg, f"{p}.mlp")
            self.mlp_norm = RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, dt)
        elif mlp_kind == LAYER_MOE:
            from .qwen3_moe import MoEBlock
            self.mlp = MoEBlock(cfg, f"{p}.mlp")
            self.mlp_norm = RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, dt)
        else:
            self.mlp = None

    def forward(self, h, residual, meta, cache, cos_sin, comm):
        if self.mixer is not None:
            if residual is None:
                residual = h
                x = self.norm(h)
            else:
                x, residual = comm.add_rmsnorm(h, residual, self.norm.weight, self.norm.eps)
            if self.kind == LAYER_ATTENTION:
                h = self.mixer(x, meta, cache.kv_layer(self.idx), cos_sin)
            else:
                h = self.mixer(x, meta, cache.recurrent, self.idx)
        if self.mlp is not None:
            if residual is None:
                residual = h
                x = self.mlp_norm(h)
            else:
                x, residual = comm.add_rmsnorm(h, residual, self.mlp_norm.weight, self.mlp_norm.eps)
            h = self.mlp(x)
        return h, residual


class HybridTransformer(nn.Module):
    def __init__(self, cfg: ModelConfig):
        super().__init__()
        self.cfg = cfg
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=cfg.compute_dtype)
        self.embed_tokens.weight.requires_grad_(False)
        self.layers = nn.ModuleList([HybridLayer(cfg, i) for i in range(cfg.num_hidden_layers)])
        self.norm = RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, cfg.compute_dtype)

    def forward(self, ids, meta, cache, cos_sin, comm, inputs_embeds=None, capture_layers=()):
        h = ops.embedding(ids, self.embed_tokens.weight) if inputs_embeds is None else inputs_embeds
        residual = None
        taps = []
        for i, layer in enumerate(self.layers):
            h, residual = layer(h, residual, meta, cache, cos_sin, comm)
            if i in capture_layers:
                taps.append((h.float() + residual.float()).to(h.dtype) if comm.world_size == 1 else comm.all_reduce(h).add_(residual))
        x, _ = comm.add_rmsnorm(h, residual, self.norm.weight, self.norm.eps)
        return (x, taps) if capture_layers else x


@register_model("nemotron_h", "nemotron_h_hybrid", "qwen3_next", "qwen3_5")
class HybridCausalLM(CausalLM):
    transformer_cls = HybridTransformer
    needs_cache_set = True      # forward takes the cache manager (KV + recurrent pools), not the bare KV pool

    @torch.no_grad()
    def replay_recurrent(self, record: dict, rows: torch.Tensor, meta: StepMeta, cache) -> int:
        """Advance the recurrent state of every Mamba / DeltaNet layer over the recorded kernel inputs of ``rows`` (row indices into
        the recorded step, grouped by sequence as ``meta`` describes).  The caller has restored the state rows of those sequences
        to what they were before the recorded step.  Returns the number of layers replayed.  This is the commit of a partly
        accepted draft chain on a hybrid target: two small kernels per recurrent layer instead of a second pass through the
        whole model (the reference's per-layer replay data, ``cpp/runtime/commitPolicy``, ``mtpStateScatterKernels``)."""
        n = 0
        for layer in self.model.layers:
            if layer.kind in (LAYER_MAMBA, LAYER_GDN) and layer.idx in record:
                layer.mixer.replay(record[layer.idx], rows, meta, cache.recurrent, layer.idx)
                n += 1
        return n
