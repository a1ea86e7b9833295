"""Operator front end.

Each function executes the hand-written sm_100a kernel when its tensors live on a CUDA
device and the plain-PyTorch statement (``ops.reference``) on CPU.  There is no silent
fallback on a GPU: if the native library is missing, the CUDA path raises.

Parity: the custom-op surface of ``tensorrt_edgellm/models/ops.py`` (attention_plugin :145,
nvfp4 ops :917-951, causal_conv1d :1541, update_ssm_state :1631, gated_delta_net :1908,
MoE plugins :2017-2209, all_reduce :2754) expressed as directly executable functions.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import reference as ref
from .meta import StepMeta, build_step_meta

__all__ = ["StepMeta", "build_step_meta", "ref", "cuda_ops"]


def cuda_ops():
    """The ctypes binding module (imported lazily so CPU-only use never touches it)."""
    from . import cuda as _cuda
    return _cuda


def rmsnorm(x, weight, eps):
    if x.is_cuda:
        return cuda_ops().rmsnorm(x, weight, eps)
    return ref.rmsnorm(x, weight, eps)


def add_rmsnorm(x, residual, weight, eps, quant_scale=None):
    """``quant_scale`` (CUDA only): emit the normalised output directly as NVFP4 for the next GEMM."""
    if x.is_cuda:
        if quant_scale is not None:
            return cuda_ops().rmsnorm_quant(x, residual, weight, eps, quant_scale)
        return cuda_ops().add_rmsnorm(x, residual, weight, eps)
    return ref.add_rmsnorm(x, residual, weight, eps)


def rmsnorm_maybe_quant(x, weight, eps, quant_scale=None):
    if x.is_cuda and quant_scale is not None:
        return cuda_ops().rmsnorm_quant(x, None, weight, eps, quant_scale)[0]
    return rmsnorm(x, weight, eps)


def layernorm(x, weight, bias, eps):
    if x.is_cuda:
        return cuda_ops().layernorm(x, weight, bias, eps)
    return ref.layernorm(x, weight, bias, eps)


def gated_group_rmsnorm(x, z, weight, n_groups, eps):
    if x.is_cuda:
        return cuda_ops().gated_group_rmsnorm(x, z, weight, n_groups, eps)
    return ref.gated_group_rmsnorm(x, z, weight, n_groups, eps)


def swiglu(gate_up, quant_scale=None, interleaved=False):
    """``interleaved``: the columns hold blocks of 64 gate features followed by their 64 up features (the layout the fused
    gate/up GEMM epilogue uses) instead of ``[gate | up]``; only the quantising CUDA form takes it."""
    if gate_up.is_cuda:
        if quant_scale is not None:
            return cuda_ops().swiglu_quant(gate_up, quant_scale, interleaved)
        assert not interleaved
        return cuda_ops().swiglu(gate_up)
    assert not interleaved
    return ref.swiglu(gate_up)


def geglu(gate_up, tanh_approx=True):
    """``gelu(gate) * up`` over the fused ``[T, 2·I]`` projection output (GeGLU MLPs)."""
    if gate_up.is_cuda:
        return cuda_ops().geglu(gate_up, tanh_approx)
    inter = gate_up.shape[-1] // 2
    g = torch.nn.functional.gelu(gate_up[..., :inter].float(), approximate="tanh" if tanh_approx else "none")
    return (g * gate_up[..., inter:].float()).to(gate_up.dtype)


def glu(gate_up, act="gelu_tanh"):
    """``act(gate) * up`` over the fused ``[T, 2·I]`` projection output; ``act``: ``"gelu_tanh"``, ``"relu"`` or ``"silu"``."""
    if act == "gelu_tanh":
        return geglu(gate_up, True)
    if act == "silu":
        if gate_up.is_cuda and gate_up.dtype == torch.float32:
            return cuda_ops().clamped_glu(gate_up, 0.0, 1.0, up_offset=0.0)
        return swiglu(gate_up)
    if act != "relu":
        raise ValueError(f"unknown gate activation {act!r}")
    if gate_up.is_cuda:
        return cuda_ops().reglu(gate_up)
    inter = gate_up.shape[-1] // 2
    return (torch.relu(gate_up[..., :inter].float()) * gate_up[..., inter:].float()).to(gate_up.dtype)


def xielu(x, coef):
    """``coef[0] x² + x / 2`` above zero, ``coef[1] (exp(x) - 1 - x) + x / 2`` below; ``coef`` fp32 ``[2]``."""
    if x.is_cuda:
        return cuda_ops().xielu(x, coef)
    return ref.xielu(x, coef)


def softcap_(logits, cap):
    """``cap * tanh(logits / cap)`` of fp32 logits, in place."""
    if logits.is_cuda:
        return cuda_ops().softcap_(logits, cap)
    return logits.div_(cap).tanh_().mul_(cap)


def relu2(x):
    if x.is_cuda:
        return cuda_ops().relu2(x)
    return ref.relu2(x)


def gelu(x, tanh_approx=False):
    if x.is_cuda:
        return cuda_ops().gelu(x, tanh_approx)
    return torch.nn.functional.gelu(x.float(), approximate="tanh" if tanh_approx else "none").to(x.dtype)


def embedding(ids, table):
    if hasattr(table, "lookup"):              # FP8 / NVFP4 table (models/embedding.py): gather stored rows, then expand
        return table.lookup(ids)
    if table.is_cuda:
        return cuda_ops().embedding(ids, table)
    return ref.embedding(ids, table)


def linear(x, weight, bias=None):
    if x.is_cuda:
        return cuda_ops().gemm(x, weight, bias)
    return ref.linear(x, weight, bias)


def rope_kv_write(qkv, kv_layer, meta, cos_sin, num_q_heads, num_kv_heads, head_dim,
                  q_norm_w=None, k_norm_w=None, eps=1e-6):
    if qkv.is_cuda:
        return cuda_ops().rope_kv_write(qkv, kv_layer, meta, cos_sin, num_q_heads, num_kv_heads, head_dim,
                                        q_norm_w, k_norm_w, eps)
    return ref.rope_kv_write(qkv, kv_layer, meta, cos_sin, num_q_heads, num_kv_heads, head_dim,
                             q_norm_w, k_norm_w, eps)


def rope_cos_sin(max_pos, rotary_dim, theta, scaling=None, device="cpu", pairs=0):
    """RoPE ``[max_pos, rotary_dim]`` cos | sin table (fp32, angles in fp64) with the frequency scaling of the checkpoint; built by
    a kernel when the table lives on a GPU.  ``pairs`` > ``rotary_dim / 2``: the table goes on to that many pairs, of angle zero."""
    dev = torch.device(device)
    if dev.type == "cuda":
        inv, att = ref.rope_frequencies(max_pos, rotary_dim, theta, scaling)
        if pairs:
            inv = torch.nn.functional.pad(inv, (0, pairs - inv.numel()))
        return cuda_ops().rope_table(inv, att, max_pos, dev)
    t = ref.rope_cos_sin(max_pos, rotary_dim, theta, scaling, device=device)
    if pairs:
        c, s = t.chunk(2, dim=-1)
        fill = pairs - c.shape[-1]
        t = torch.cat([torch.nn.functional.pad(c, (0, fill), value=1.0), torch.nn.functional.pad(s, (0, fill))], dim=-1)
    return t


def mrope_rows(cos_sin, positions3, sections):
    """Multimodal RoPE: per-row cos | sin tables gathered by each row's (temporal, height, width) positions."""
    if cos_sin.is_cuda:
        return cuda_ops().mrope_rows(cos_sin, positions3, sections)
    return ref.mrope_rows(cos_sin, positions3, sections)


def rope_q(q, kv_layer, meta, cos_sin, num_q_heads, head_dim, q_norm_w=None, eps=1e-6):
    """Per-head RMSNorm and RoPE of the queries of a layer that writes no keys / values (``kv_layer`` is only read later; the
    GPU form runs the RoPE + KV-write kernel with zero KV heads, so nothing is stored)."""
    if q.is_cuda:
        return cuda_ops().rope_kv_write(q, kv_layer, meta, cos_sin, num_q_heads, 0, head_dim, q_norm_w, None, eps)
    return ref.rope_q(q, meta, cos_sin, num_q_heads, head_dim, q_norm_w, eps)


def paged_attention(q, kv_layer, meta, scale, sliding_window=None, sinks=None, causal=True, chunk=0, fp32_weights=False, back=None, out=None):
    """``chunk`` > 0: row at position ``i`` sees only keys ``j`` with ``j // chunk == i // chunk`` (and ``j <= i``).
    ``fp32_weights``: the softmax weights keep fp32 precision in the weighted sum of 16-bit values.
    ``back``: ``(cos | sin table, factor)``; every output is turned back by its position (neighbouring features form the pairs) and
    multiplied, before it is rounded.  ``out``: where the rows go (``[T, heads * head]``, its rows may lie further apart)."""
    if q.is_cuda:
        return cuda_ops().paged_attention(q, kv_layer, meta, scale, sliding_window, sinks, causal=causal, chunk=chunk, fp32_weights=fp32_weights,
                                          back=back, out=out)
    o = ref.paged_attention(q, kv_layer, meta, scale, sliding_window, sinks, causal=causal, chunk=chunk, back=back)
    return o if out is None else out.copy_(o.reshape(out.shape))


def linear_f32(x, weight, bias=None):
    """``x · weightᵀ (+ bias)`` with the fp32 sums as the result."""
    if x.is_cuda:
        return cuda_ops().gemm_f32out(x, weight, bias)
    y = x.float() @ weight.float().t()
    return y if bias is None else y + bias.float()


def stream_norm(stream, weight, eps, *, delta=None, routed=None, mult=1.0, step=None, offset=0.0, ids=None, table=None, dtype=None,
                alpha=None, bias=None, table_mult=1.0):
    """Advance the fp32 residual stream and normalise it for the next layer: returns ``(stream, h)``.

    ``stream`` (or ``table[ids] * table_mult`` when it is ``None``) ``+ mult * (delta + routed) + step``; ``h`` is its RMS norm times
    ``offset + weight`` in the activation type (``None`` without ``weight``), or, with a scalar ``alpha``, the element-wise
    ``tanh(alpha * x) * weight + bias``.  ``routed`` is a mixture block's output: a dense tensor, or
    :class:`models.qwen3_moe.RoutedRows`, whose weighted sum the kernel takes itself."""
    t = ids if stream is None else stream
    args = (stream, weight, eps, delta, routed, mult, step, offset, ids, table, dtype, alpha, bias, table_mult)
    if t.is_cuda:
        return cuda_ops().stream_norm(*args)
    return ref.stream_norm(*args)


@dataclass
class Bigram:
    """Second embedding of a token: row ``(previous * mul_prev + token * mul_cur) mod buckets`` of ``table``, row ``buckets`` where a
    sequence starts.  ``last``: ``[seats, 1]`` int32, the last token of every sequence."""

    table: torch.Tensor
    last: torch.Tensor
    buckets: int
    mul_prev: int
    mul_cur: int


def stream_post(stream, delta, weight, groups, eps, meta, dtype, *, ids=None, table=None, bigram=None, conv=None, history=None, out_norm=None, sums=None):
    """Advance the fp32 residual stream by a normed sublayer output and write what the next sublayer reads: ``(stream, h)``.

    ``stream`` (or ``table[ids]`` plus the row of ``bigram`` when it is ``None``) ``+ norm(delta) * weight``; the norm divides each of ``groups``
    equal parts of a row by its own root mean square.  ``sums``: ``(partial sums of squares [T, n], features)`` of the row that was projected
    to ``delta``, which still has to be divided by that row's root mean square.  ``h`` in ``dtype`` is the stream itself; with ``conv`` ``[taps, width]`` (fp32) the
    stream plus its causal convolution over time, whose ``history`` ``[seats, taps - 1, width]`` (fp32) is advanced; with ``out_norm`` the norm
    of the stream times that weight."""
    t = ids if stream is None else stream
    f = cuda_ops().stream_post if t.is_cuda else ref.stream_post
    return f(stream, delta, weight, groups, eps, meta, dtype, ids, table, bigram, conv, history, out_norm, sums)


def stream_sandwich(stream, eps, meta, dtype, *, ids=None, table=None, positions=None, delta=None, routed=None, post=None, mult=1.0, norm=None,
                    shift=None, state=None):
    """The fp32 residual stream of blocks with a norm in front of and behind every sublayer: ``(stream, h)``.

    ``stream`` (or ``table[ids]`` when it is ``None``), plus the row of ``positions`` of every token's position when given, ``+ mult * rms_norm(delta
    + routed) * post``; ``h`` in ``dtype`` is its RMS norm times ``norm``.  ``shift`` ``[width]``: features of ``h`` move by these shares towards
    the row before it in its sequence; ``state`` ``[seats, 1, width]`` (fp32) holds the last normed row of every sequence and is
    advanced.  ``routed``: a dense tensor, or :class:`models.qwen3_moe.RoutedRows`, whose weighted sum the kernel takes itself."""
    t = ids if stream is None else stream
    f = cuda_ops().stream_sandwich if t.is_cuda else ref.stream_sandwich
    return f(stream, eps, meta, dtype, ids, table, positions, delta, routed, post, mult, norm, shift, state)


def lightning(rows, norm_w, powers, state, meta):
    """Linear attention with a constant decay per head over packed ``[q | k | v | g]`` rows: silu on q, k and v, the recurrence, weight and
    sigmoid gate.  Returns ``(u [T, heads · dv], sums [T, heads · dv / 32])``: the gated read-outs before the RMS norm over all heads of a
    row, and sums of squares of the read-outs; the norm's division commutes with the output projection and is left to the consumer
    (:func:`stream_post`).  ``powers`` ``[heads, n + 1]``: powers of the decays from 0 on; ``state`` ``[seats, heads, dk, dv]`` is
    advanced in place."""
    f = cuda_ops().lightning if rows.is_cuda else ref.lightning
    return f(rows, norm_w, powers, state, meta)


def moe_route_chosen(logits, top_k):
    """The ``top_k`` largest fp32 logits per row and the softmax over them: ``(weights, indices)``."""
    if logits.is_cuda:
        return cuda_ops().moe_route_chosen(logits, top_k)
    return ref.moe_route_chosen(logits, top_k)


def moe_route_sigmoid_groups(logits, correction, top_k, groups, keep, scale):
    """Scores ``sigmoid(logits)``; the ``top_k`` largest ``score + correction`` inside the ``keep`` best of ``groups`` equal groups of neighbours (a
    group's worth: the sum of its two largest).  Returns ``(scale * scores, indices)`` of the chosen."""
    if logits.is_cuda:
        return cuda_ops().moe_route_softmax_topk(logits, top_k, False, correction, True, groups, keep, scale)
    return ref.moe_route_sigmoid_group_topk(logits, correction, top_k, groups, keep, False, scale)


def mlstm(qkvg, gates, norm_w, state, norm_state, meta, scale, cap, eps, dv_real):
    """Matrix-memory LSTM over packed ``[q | k | v | g]`` rows with head norm and output gate: ``[T, heads · dv]``.  ``state``
    ``[seats, heads, dk, dv]`` and ``norm_state`` ``[seats, heads, dk + 1]`` (normaliser, running maximum) are advanced in place."""
    if qkvg.is_cuda:
        return cuda_ops().mlstm(qkvg, gates, norm_w, state, norm_state, meta, scale, cap, eps, dv_real)
    return ref.mlstm(qkvg, gates, norm_w, state, norm_state, meta, scale, cap, eps, dv_real)


def channel_delta(qkv, decay, gate, beta, conv_w, a_log, decay_bias, norm_w, conv_state, state, meta, spec, eps, out=None, mult=1.0):
    """Delta-rule mixer with a decay per key channel (or per head), from packed projections to gated head outputs ``[T, heads * v_pad]``
    times ``mult``.

    ``qkv``: packed ``[q | k | v]`` rows of padded heads; ``decay`` (fp32, before bias and softplus; ``[T, heads]`` with one decay per
    head), ``gate`` and ``beta`` (fp32) are pre-activations.  ``conv_state`` ``[seats, channels, taps - 1]`` and ``state``
    ``[seats, heads, k_pad, v_pad]`` are advanced in place.  ``spec``: :class:`config.ChannelDeltaConfig`.  ``out``: where the rows go."""
    f = cuda_ops().channel_delta if qkv.is_cuda else ref.channel_delta
    return f(qkv, decay, gate, beta, conv_w, a_log, decay_bias, norm_w, conv_state, state, meta, spec, eps, out=out, mult=mult)


def query_temperature(length, coef, every, device="cpu"):
    """``[length]`` fp32 factors ``1 + coef * ln(floor((position + 1) / every) + 1)``."""
    return ref.query_temperature(length, coef, every, device)


def unit_kv_write(qkv, kv_layer, meta, temperature, num_q_heads, num_kv_heads, head_dim, real_dim, eps):
    """Queries and keys over their root mean square (``real_dim`` features of a padded head), queries times the temperature of their
    position; writes keys and values into the paged cache and returns ``q [T, Hq, D]``."""
    f = cuda_ops().unit_kv_write if qkv.is_cuda else ref.unit_kv_write
    return f(qkv, kv_layer, meta, temperature, num_q_heads, num_kv_heads, head_dim, real_dim, eps)


def turned_kv_write(rows, kv_layer, meta, key_table, value_table, q_norm, k_norm, spec, eps):
    """Packed q | k | v rows: RMS norms over all heads of the queries and of the keys, interleaved rotation of both by ``key_table`` and of the
    values by ``value_table`` (cos | sin, a pair per two padded features); keys and values go to the paged cache.  Returns ``q [T, Hq, D]``.
    ``spec``: :class:`config.AttentionConfig`."""
    f = cuda_ops().turned_kv_write if rows.is_cuda else ref.turned_kv_write
    return f(rows, kv_layer, meta, key_table, value_table, q_norm, k_norm, spec, eps)


def mixed_kv_write(rows, kv_layer, meta, mix, first, share, spec):
    """Packed q | k | v rows (and what lies behind them) of padded heads: keys go to the paged cache, values too, ``(1 - share) v + share *
    first`` when ``first`` ``[T, kv heads * its pad]`` is given (its heads may be padded to another size).  Returns the wide queries: head ``h`` holds, for every KV head ``c``, the sum of
    ``mix[h, g] q_g`` over the query heads ``g`` of ``c``.  ``spec``: :class:`config.AttentionConfig`."""
    f = cuda_ops().mixed_kv_write if rows.is_cuda else ref.mixed_kv_write
    return f(rows, kv_layer, meta, mix, first, share, spec)


def mixed_attention(q, kv_layer, meta, slopes, gate, spec):
    """Windowed attention of wide queries (see :func:`mixed_kv_write`) over the keys of all KV heads at once; head ``h`` loses ``slopes[h]`` times
    the distance and reads the values of its own KV head; heads times ``sigmoid(gate)`` (``[T, heads * pad]``, or None).  ``[T, heads * pad]``."""
    f = cuda_ops().mixed_attention if kv_layer.is_cuda else ref.mixed_attention
    return f(q, kv_layer, meta, slopes, gate, spec)


def latent_write(rows, kv_layer, meta, cos_sin, norm_w, spec, eps):
    """Packed ``[q unrotated | q rotated part | latent | rotated key part]`` rows: RMS norm of the latent, interleaved rotation of the
    rotated parts, and ``[latent | key part]`` written to the paged cache ``[pages, 1, 1, P, row]``.  Returns the rows with their query
    columns ready (modified in place)."""
    f = cuda_ops().latent_write if rows.is_cuda else ref.latent_write
    return f(rows, kv_layer, meta, cos_sin, norm_w, spec, eps)


def latent_attention(rows, kv_layer, meta, kv_up, key_up_t, spec):
    """Causal attention of the queries in ``rows`` (see :func:`latent_write`) over cached latents: ``[T, heads * v_pad]``.

    ``kv_up`` ``[heads * k_pad + heads * v_pad, rank_pad]`` expands a latent into keys and values; ``key_up_t``
    ``[heads, rank_pad, k_pad]`` is its key part with exchanged axes."""
    f = cuda_ops().latent_attention if rows.is_cuda else ref.latent_attention
    return f(rows, kv_layer, meta, kv_up, key_up_t, spec)


def kv_fp8_prepare(kv_layer, meta, scales, dtype, window=0):
    """FP8 KV layer → the 16-bit staging layer holding the step's cached pages (new rows are written into it next)."""
    if kv_layer.is_cuda:
        cu = cuda_ops()
        stage = cu.kv_fp8_stage(kv_layer, dtype)
        cu.kv_fp8_load(kv_layer, stage, meta, scales, window)
        return stage
    stage = torch.zeros(kv_layer.shape, dtype=dtype)
    ref.kv_fp8_load(kv_layer, stage, meta, scales, window)
    return stage


def kv_fp8_commit(kv_layer, stage, meta, scales):
    """Quantise the step's new rows from the staging layer into the FP8 layer (and round the staged rows the same way)."""
    if kv_layer.is_cuda:
        return cuda_ops().kv_fp8_store(kv_layer, stage, meta, scales)
    return ref.kv_fp8_store(kv_layer, stage, meta, scales)


def argmax(logits):
    if logits.is_cuda:
        return cuda_ops().argmax(logits)
    return ref.argmax(logits)


def sample(logits, temperature, top_k, top_p, uniforms):
    if logits.is_cuda:
        return cuda_ops().sample(logits, temperature, top_k, top_p, uniforms)
    return ref.sample(logits, temperature, top_k, top_p, uniforms)


def moe_route(logits, top_k, renormalize=True):
    if logits.is_cuda:
        return cuda_ops().moe_route_softmax_topk(logits, top_k, renormalize)
    return ref.moe_route_softmax_topk(logits, top_k, renormalize)


def causal_conv1d(x, weight, bias, conv_state, meta, activation=True):
    if x.is_cuda:
        return cuda_ops().causal_conv1d(x, weight, bias, conv_state, meta, activation)
    return ref.causal_conv1d(x, weight, bias, conv_state, meta, activation)


def ssm_scan(x, dt, A, B, C, D, dt_bias, ssm_state, meta, z=None, dt_softplus=True, dt_limit=0.0):
    if x.is_cuda:
        return cuda_ops().ssm_scan(x, dt, A, B, C, D, dt_bias, ssm_state, meta, z, dt_softplus, dt_limit)
    return ref.ssm_scan(x, dt, A, B, C, D, dt_bias, ssm_state, meta, z, dt_softplus, dt_limit)


def gated_delta_rule(q, k, v, a, b, A_log, dt_bias, state, meta):
    if q.is_cuda:
        return cuda_ops().gated_delta_rule(q, k, v, a, b, A_log, dt_bias, state, meta)
    return ref.gated_delta_rule(q, k, v, a, b, A_log, dt_bias, state, meta)


def spec_accept_greedy(target_tokens, tree_tokens, parents, max_path, force_len=0):
    if tree_tokens.is_cuda:
        return cuda_ops().spec_accept_greedy(target_tokens, tree_tokens, parents, max_path, force_len)
    return ref.spec_accept_greedy(target_tokens, tree_tokens, parents, max_path, force_len)


def token_logprobs(logits, tokens, k):
    """Log-probability of each row's token and its ``k`` most likely tokens: ``(chosen, top_ids, top_values)``."""
    if logits.is_cuda and logits.stride(-1) == 1 and k <= 32 and logits.dtype in (torch.float16, torch.bfloat16, torch.float32):
        return cuda_ops().token_logprobs(logits, tokens, k)
    return ref.token_logprobs(logits, tokens, k)


def spec_accept_sampling(target_probs, tree_tokens, parents, max_path, uniforms):
    """Lossless acceptance along a draft tree for sampled requests (sibling-by-sibling rejection against each node's target
    distribution, bonus token from the residual): ``(path, path_len, bonus)``."""
    if target_probs.is_cuda:
        return cuda_ops().spec_accept_sampling(target_probs, tree_tokens, parents, max_path, uniforms)
    return ref.spec_accept_sampling(target_probs, tree_tokens, parents, max_path, uniforms)


def eagle_tree_meta(parents, base_pos, depth_base, pos_offset):
    """``(mask [B*R, W], depth [B, R], positions [B*R])`` of a batch of trees given as parent tables."""
    if parents.is_cuda:
        return cuda_ops().eagle_tree_meta(parents, base_pos, depth_base, pos_offset)
    return ref.eagle_tree_meta(parents, base_pos, depth_base, pos_offset)


def eagle_select_verify(p_sc, p_tok, p_par, p_dep, root, keep):
    """Verification tree ``(tokens, parents, depths)``: the ``keep`` best pool candidates in pool order behind the root."""
    if p_sc.is_cuda:
        return cuda_ops().eagle_select_verify(p_sc, p_tok, p_par, p_dep, root, keep)
    return ref.eagle_select_verify(p_sc, p_tok, p_par, p_dep, root, keep)


def dflash2_grouped_dynamic_conv(hidden, delta, base, residual, block, group_size):
    """``out[t, c] = Σ_k (base[k, c] + delta[t, k, c // group_size]) · hidden[t - k, c]`` over the taps that stay inside row ``t``'s
    proposal block, plus ``residual`` when given."""
    if hidden.is_cuda and hidden.dtype in (torch.float16, torch.bfloat16) and group_size % 2 == 0 and base.shape[0] <= 4:
        return cuda_ops().dflash2_grouped_dynamic_conv(hidden, delta, base, residual, block, group_size)
    return ref.dflash2_grouped_dynamic_conv(hidden, delta, base, residual, block, group_size)


def dflash2_selector_walk(cand_ids, unary, projected, anchor, pred_codebook, succ_codebook, temperatures=None, uniforms=None):
    """Chain selector of DFlash 2: per slot, the candidate with the best ``unary + <P[prev] ⊙ z, Q[candidate]>`` (or a draw from
    the softmax of those scores) becomes the slot's token and the next slot's predecessor."""
    if (cand_ids.is_cuda and projected.dtype in (torch.float16, torch.bfloat16) and pred_codebook.dtype == projected.dtype
            and succ_codebook.dtype == projected.dtype and cand_ids.shape[-1] <= 32 and projected.shape[-1] <= 1024):
        return cuda_ops().dflash2_selector_walk(cand_ids, unary, projected, anchor, pred_codebook, succ_codebook, temperatures, uniforms)
    return ref.dflash2_selector_walk(cand_ids, unary, projected, anchor, pred_codebook, succ_codebook, temperatures, uniforms)


def markov_chain_propose(logits, w1, w2, first_prev, temperatures=None, uniforms=None):
    """DSpark's Markov head: step ``i`` picks from ``logits[:, i] + W2 · W1[previous token]``.  All-greedy batches run as one
    fused correction + arg-max kernel per step on the GPU; batches with sampled rows use library ops."""
    if (logits.is_cuda and temperatures is None and w1.dtype in (torch.float16, torch.bfloat16) and w2.dtype == w1.dtype
            and w1.shape[1] <= 512 and logits.shape[0] * w1.shape[1] <= 48 * 1024 and w2.shape[0] == logits.shape[-1]):
        return cuda_ops().markov_greedy_chain(logits, w1, w2, first_prev)
    return ref.markov_chain_propose(logits, w1, w2, first_prev, temperatures, uniforms)


def lattice_chain_walk(cand_ids, transition, temperatures=None, uniforms=None):
    """LiLiCorr's walk: per slot, the candidate with the best ``transition[slot, previous index, ·]`` (or a draw from its softmax)."""
    if cand_ids.is_cuda and cand_ids.shape[-1] <= 32:
        return cuda_ops().lattice_chain_walk(cand_ids, transition, temperatures, uniforms)
    return ref.lattice_chain_walk(cand_ids, transition, temperatures, uniforms)


def low_rank_candidate_head(hidden, down_proj, up_proj, lm_head, num_candidates):
    """EAGLE-4 candidate head: ``(ids [R, Kc] int32, log-probabilities [R, Kc] fp32)`` of the ``Kc`` tokens the low-rank
    scores pick, ordered by their exact logits.  On the GPU the two low-rank products and the top-k are library ops and the
    exact rescoring, ordering and log-softmax are one kernel."""
    if hidden.is_cuda and hidden.dtype in (torch.float16, torch.bfloat16) and lm_head.dtype == hidden.dtype:
        proj = (hidden @ down_proj.to(hidden.dtype).t())                  # fp32 accumulation, rounded to the 16-bit type
        scores = (proj @ up_proj.to(hidden.dtype).t()).float()
        scores = torch.nan_to_num(scores, nan=float("-inf"))
        cand = scores.topk(num_candidates, dim=-1).indices
        return cuda_ops().candidate_rescore(hidden, lm_head, cand)
    return ref.low_rank_candidate_head(hidden, down_proj, up_proj, lm_head, num_candidates)


def kv_commit_path(pool, page_table, past_len, path, path_len):
    if pool.is_cuda:
        return cuda_ops().kv_commit_path(pool, page_table, past_len, path, path_len)
    return ref.kv_commit_path(pool, page_table, past_len, path, path_len)


def apply_token_bitmask(logits, bitmask):
    """Entries whose bit is 0 in ``bitmask [rows, ceil(V/32)]`` become very negative (guided decoding)."""
    if logits.is_cuda:
        return cuda_ops().apply_token_bitmask(logits, bitmask)
    return ref.apply_token_bitmask(logits, bitmask)


def ddtree_candidates(logits, k):
    """Per-depth top-``k`` candidates of a block draft with whole-vocabulary log-probabilities (torch ops on the logits' device)."""
    return ref.ddtree_candidates(logits, k)


def ddtree_assemble(cand_ids, cand_lp, root_tokens, num_nodes, depth_confidence=None, survival_threshold=0.0):
    """Best-first verification tree from per-depth candidates.  A few dozen nodes per sequence: assembled on the host from the
    candidate lists (one small device→host copy), results returned on the candidates' device."""
    return ref.ddtree_assemble(cand_ids, cand_lp, root_tokens, num_nodes, depth_confidence, survival_threshold)
