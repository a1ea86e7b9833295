"""ctypes binding of the native sm_100a kernel library (``_lib/libtelb_kernels.so``).

Kernels are launched on the current torch CUDA stream with raw device pointers, so they are
captured by ``torch.cuda.graph`` like any other launch.  A missing or stale library is an error:
nothing in this module falls back to PyTorch on a GPU.
"""
from __future__ import annotations

import ctypes
import os
import threading
from typing import Dict, Optional, Tuple

import torch

from .meta import StepMeta

_LIB_PATH = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "_lib", "libtelb_kernels.so")
_lib: Optional[ctypes.CDLL] = None
KERNEL_FAMILY = ""       # a family whose own kernel library (build.KERNEL_SETS) serves this process when the whole one is not built

c_int, c_ll, c_float, c_vp = ctypes.c_int, ctypes.c_longlong, ctypes.c_float, ctypes.c_void_p


def lib() -> ctypes.CDLL:
    global _lib
    if _lib is None:
        # fault-injection hook for tests of the failure path (the reference's TRT_EDGELLM_TEST_FAIL_CUTEDSL_MODULE,
        # cpp/kernels/cuteDslModuleLoader.cpp:178): the named library "fails to load" deterministically
        if os.environ.get("TELB_TEST_FAIL_KERNEL_LIBRARY", "") in ("1", os.path.basename(_LIB_PATH)):
            raise RuntimeError(f"native kernel library {_LIB_PATH} failed to load (TELB_TEST_FAIL_KERNEL_LIBRARY is set)")
        if KERNEL_FAMILY and not os.path.exists(_LIB_PATH):
            from ..build import kernel_library
            _lib = ctypes.CDLL(kernel_library(KERNEL_FAMILY))
            _lib.telb_last_error.restype = ctypes.c_char_p
            return _lib
        if not os.path.exists(_LIB_PATH):
            raise RuntimeError(f"native kernel library not built: {_LIB_PATH} (run `python -m tensorrt_edge_llm_b200.build`)")
        _lib = ctypes.CDLL(_LIB_PATH)
        _lib.telb_last_error.restype = ctypes.c_char_p
    return _lib


LAUNCHES = 0      # kernels of this library launched (or captured) so far in this process


_DEBUG_SYNC = os.environ.get("TELB_DEBUG_SYNC", "0") == "1"     # synchronise after every op so a device error names its op


# Tensors whose pointers were taken for the launch being assembled.  A converted temporary (``x.to(int32)`` written inline
# in an argument list) would otherwise be freed as soon as its pointer is extracted, and the caching allocator may hand the
# same bytes to the next inline conversion of the same call, before the kernel has been enqueued.
_KEEP = threading.local()


def _check(rc: int, what: str, n: int = 1) -> None:
    global LAUNCHES
    held = getattr(_KEEP, "tensors", None)
    if held:
        held.clear()                      # the launch is enqueued: stream order protects the memory from here on
    if rc != 0:
        raise RuntimeError(f"{what} failed: {lib().telb_last_error().decode()}")
    LAUNCHES += n
    if _DEBUG_SYNC and not torch.cuda.is_current_stream_capturing():
        try:
            torch.cuda.synchronize()
        except RuntimeError as e:
            raise RuntimeError(f"device error surfaced after {what}: {e}") from None


def _p(t: Optional[torch.Tensor]):
    if t is None:
        return c_vp(0)
    if not t.is_cuda:        # a host pointer handed to a kernel is a device fault, not an exception
        raise ValueError(f"kernel argument of shape {tuple(t.shape)} lives on {t.device}, not on the GPU")
    held = getattr(_KEEP, "tensors", None)
    if held is None:
        held = _KEEP.tensors = []
    if len(held) > 4096:                  # pointers taken outside a _check-wrapped call must not accumulate
        held.clear()
    held.append(t)
    return c_vp(t.data_ptr())


def _stream() -> c_vp:
    return c_vp(torch.cuda.current_stream().cuda_stream)


def _is_bf16(t: torch.Tensor) -> int:
    if t.dtype == torch.bfloat16:
        return 1
    if t.dtype == torch.float16:
        return 0
    raise TypeError(f"CUDA kernels take fp16 / bf16 activations, got {t.dtype}")


def _dtype_code(t: torch.Tensor) -> int:
    """0 fp16, 1 bf16, 2 fp32: the kernels that also run in 32 bits."""
    return 2 if t.dtype == torch.float32 else _is_bf16(t)


class Workspace:
    """Per-device scratch shared by kernels that need it: split-K partial tiles and their tile
    counters (GEMM), split-KV partials (attention) and the status word every bounded wait reports
    to.  Sized once; kernels fall back to un-split execution when a problem does not fit."""

    _by_device: Dict[int, "Workspace"] = {}

    def __init__(self, device: torch.device, gemm_bytes: int = 64 << 20, attn_floats: int = 32 << 20):
        self.gemm_ws = torch.empty(gemm_bytes, dtype=torch.uint8, device=device)
        self.counters = torch.zeros(8192, dtype=torch.int32, device=device)
        self.attn_ws = torch.empty(attn_floats, dtype=torch.float32, device=device)
        self.status = torch.zeros(4, dtype=torch.int32, device=device)
        self.argmax_keys = torch.zeros(256, dtype=torch.int64, device=device)
        self.argmax_counters = torch.zeros(256, dtype=torch.int32, device=device)

    @classmethod
    def get(cls, device: torch.device) -> "Workspace":
        idx = device.index if device.index is not None else torch.cuda.current_device()
        ws = cls._by_device.get(idx)
        if ws is None:
            ws = cls._by_device[idx] = Workspace(torch.device("cuda", idx))
        return ws

    def check_status(self) -> None:
        """Raise if any kernel recorded a timed-out wait (synchronises the device)."""
        code = int(self.status[0].item())
        if code != 0:
            self.status.zero_()
            names = {1: "TMA producer", 2: "MMA issuer", 3: "epilogue", 4: "peer", 5: "bad argument"}
            raise RuntimeError(f"kernel wait timed out in role: {names.get(code, code)}")


# ------------------------------------------------------------------------------------------------


def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    x = x.contiguous()
    y = torch.empty_like(x)
    rows = x.numel() // x.shape[-1]
    _check(lib().telb_rmsnorm(_p(x), c_vp(0), _p(weight), _p(y), c_vp(0), c_ll(rows), c_int(x.shape[-1]), c_float(eps),
                              c_int(_is_bf16(x)), _stream()), "rmsnorm")
    return y


def add_rmsnorm(x: torch.Tensor, residual: torch.Tensor, weight: torch.Tensor, eps: float
                ) -> Tuple[torch.Tensor, torch.Tensor]:
    x = x.contiguous()
    residual = residual.contiguous()
    y = torch.empty_like(x)
    res = torch.empty_like(x)
    rows = x.numel() // x.shape[-1]
    _check(lib().telb_rmsnorm(_p(x), _p(residual), _p(weight), _p(y), _p(res), c_ll(rows), c_int(x.shape[-1]),
                              c_float(eps), c_int(_is_bf16(x)), _stream()), "add_rmsnorm")
    return y, res


def layernorm(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    x = x.contiguous()
    y = torch.empty_like(x)
    rows = x.numel() // x.shape[-1]
    _check(lib().telb_layernorm(_p(x), _p(weight), _p(bias), _p(y), c_ll(rows), c_int(x.shape[-1]), c_float(eps), c_int(_is_bf16(x)),
                                _stream()), "layernorm")
    return y


def gated_group_rmsnorm(x, z, weight, n_groups, eps):
    x, z = x.contiguous(), z.contiguous()
    y = torch.empty_like(x)
    rows = x.numel() // x.shape[-1]
    _check(lib().telb_gated_group_rmsnorm(_p(x), _p(z), _p(weight), _p(y), c_ll(rows), c_int(x.shape[-1]),
                                          c_int(n_groups), c_float(eps), c_int(_is_bf16(x)), _stream()), "gated_group_rmsnorm")
    return y


def geglu(gate_up: torch.Tensor, tanh_approx: bool = True) -> torch.Tensor:
    rows, two = gate_up.shape
    inter = two // 2
    out = torch.empty(rows, inter, dtype=gate_up.dtype, device=gate_up.device)
    if gate_up.dtype == torch.float32:
        if not tanh_approx:
            raise TypeError("geglu: the fp32 form covers the tanh gelu only")
        _check(lib().telb_glu_f32(_p(gate_up.contiguous()), _p(out), c_ll(rows), c_int(inter), c_int(0), _stream()), "glu_f32")
        return out
    _check(lib().telb_geglu(_p(gate_up), _p(out), c_ll(rows), c_int(inter), c_int(1 if tanh_approx else 0), c_int(_is_bf16(gate_up)),
                            _stream()), "geglu")
    return out


def reglu(gate_up: torch.Tensor) -> torch.Tensor:
    """``relu(gate) * up``."""
    gate_up = gate_up.contiguous()
    rows, two = gate_up.shape
    out = torch.empty(rows, two // 2, dtype=gate_up.dtype, device=gate_up.device)
    if gate_up.dtype == torch.float32:
        _check(lib().telb_glu_f32(_p(gate_up), _p(out), c_ll(rows), c_int(two // 2), c_int(1), _stream()), "glu_f32")
    else:
        _check(lib().telb_geglu(_p(gate_up), _p(out), c_ll(rows), c_int(two // 2), c_int(2), c_int(_is_bf16(gate_up)), _stream()), "reglu")
    return out


def xielu(x: torch.Tensor, coef: torch.Tensor) -> torch.Tensor:
    x = x.contiguous()
    assert coef.dtype == torch.float32 and coef.numel() == 2
    out = torch.empty_like(x)
    _check(lib().telb_xielu(_p(x), _p(out), c_ll(x.numel()), _p(coef), c_int(_dtype_code(x)), _stream()), "xielu")
    return out


def softcap_(logits: torch.Tensor, cap: float) -> torch.Tensor:
    if logits.dtype != torch.float32 or not logits.is_contiguous():
        raise TypeError("softcap_: contiguous fp32 logits")
    _check(lib().telb_softcap(_p(logits), c_ll(logits.numel()), c_float(cap), _stream()), "softcap")
    return logits


def swiglu(gate_up: torch.Tensor) -> torch.Tensor:
    gate_up = gate_up.contiguous()
    inter = gate_up.shape[-1] // 2
    rows = gate_up.numel() // gate_up.shape[-1]
    out = torch.empty(*gate_up.shape[:-1], inter, dtype=gate_up.dtype, device=gate_up.device)
    _check(lib().telb_swiglu(_p(gate_up), _p(out), c_ll(rows), c_int(inter), c_int(_is_bf16(gate_up)), _stream()), "swiglu")
    return out


def relu2(x: torch.Tensor) -> torch.Tensor:
    x = x.contiguous()
    out = torch.empty_like(x)
    _check(lib().telb_relu2(_p(x), _p(out), c_ll(x.numel()), c_int(_is_bf16(x)), _stream()), "relu2")
    return out


def gelu(x: torch.Tensor, tanh_approx: bool = False) -> torch.Tensor:
    x = x.contiguous()
    out = torch.empty_like(x)
    _check(lib().telb_gelu(_p(x), _p(out), c_ll(x.numel()), c_int(int(tanh_approx)), c_int(_is_bf16(x)), _stream()), "gelu")
    return out


def embedding(ids: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    ids = ids.to(torch.int32).contiguous()
    out = torch.empty(ids.numel(), table.shape[1], dtype=table.dtype, device=table.device)
    _check(lib().telb_embedding(_p(ids), _p(table), _p(out), c_ll(ids.numel()), c_int(table.shape[1]),
                                c_int(table.shape[0]), c_int(_is_bf16(table)), _stream()), "embedding")
    return out


def embedding_quant(ids, data, scale, global_scale, fmt: str, out_dtype) -> torch.Tensor:
    """Gather rows of an FP8 (``data [V, H]`` E4M3, ``scale [V]`` fp32) or NVFP4 (``data [V, H / 2]``, ``scale [V, H / 16]`` E4M3,
    ``global_scale``) embedding table and expand them to ``out_dtype`` in the same kernel."""
    assert out_dtype in (torch.float16, torch.bfloat16) and fmt in ("fp8", "nvfp4")
    ids = ids.to(torch.int32).contiguous()
    hidden = data.shape[1] * (2 if fmt == "nvfp4" else 1)
    out = torch.empty(ids.numel(), hidden, dtype=out_dtype, device=data.device)
    d, sc = data.contiguous(), scale.contiguous()
    gs = None if global_scale is None else global_scale.reshape(-1).float().contiguous()
    _check(lib().telb_embedding_quant(_p(ids), _p(d), _p(sc), _p(gs), _p(out), c_ll(ids.numel()), c_int(hidden), c_int(data.shape[0]),
                                      c_int(1 if fmt == "nvfp4" else 0), c_int(int(out_dtype == torch.bfloat16)), _stream()), "embedding_quant")
    return out


def gemm(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None,
         alpha: Optional[torch.Tensor] = None, residual: Optional[torch.Tensor] = None,
         out: Optional[torch.Tensor] = None, mode: int = 0, splits: int = 0) -> torch.Tensor:
    """``out[M,N] = x[M,K] · weight[N,K]ᵀ (* alpha[N]) (+ bias[N]) (+ residual[M,N])`` on tcgen05."""
    lead = x.shape[:-1]
    x2 = x.reshape(-1, x.shape[-1])
    if not x2.is_contiguous():
        x2 = x2.contiguous()
    m, k = x2.shape
    n = weight.shape[0]
    if weight.dtype != x.dtype:
        raise TypeError(f"gemm: activation {x.dtype} and weight {weight.dtype} differ")
    if x.dtype == torch.float32:                  # true fp32 on the CUDA cores (the tensor cores have no fp32 operands)
        if alpha is not None or residual is not None:
            raise TypeError("gemm: the fp32 product takes no column scale and no residual")
        return gemm_f32out(x2, weight, bias, out).reshape(*lead, n)
    if k % 8:
        # rows must be 16-byte multiples for the TMA descriptors: zero columns up to the next multiple of 8 change nothing
        # (patch embeddings with 3 · 14 · 14 = 588 inputs are the case in practice; the padded copies are made per call)
        pad = 8 - k % 8
        x2 = torch.nn.functional.pad(x2, (0, pad))
        weight = torch.nn.functional.pad(weight, (0, pad))
        k += pad
    if out is None:
        out = torch.empty(m, n, dtype=x.dtype, device=x.device)
    ws = Workspace.get(x.device)
    _check(lib().telb_gemm_f16(_p(x2), _p(weight), _p(out), c_int(m), c_int(n), c_int(k), _p(bias), _p(alpha),
                               _p(residual), c_int(_is_bf16(x)), _p(ws.gemm_ws), c_ll(ws.gemm_ws.numel()),
                               _p(ws.counters), c_int(ws.counters.numel()), _p(ws.status), c_int(mode), c_int(splits),
                               _stream()), "gemm")
    return out.reshape(*lead, n)


def gemm_f32out(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out[M,N]`` fp32 ``= x · weightᵀ (+ bias)``: tensor-core product of 16-bit operands, or the fp32 kernel for fp32 operands.
    ``bias`` is fp32."""
    x2 = x if x.is_contiguous() else x.contiguous()
    m, k = x2.shape
    n = weight.shape[0]
    if weight.dtype != x.dtype or (bias is not None and bias.dtype != torch.float32):
        raise TypeError(f"gemm_f32out: activation {x.dtype}, weight {weight.dtype}, bias {None if bias is None else bias.dtype}")
    if out is None:
        out = torch.empty(m, n, dtype=torch.float32, device=x.device)
    if x.dtype == torch.float32:
        _check(lib().telb_gemm_f32(_p(x2), _p(weight), _p(out), c_int(m), c_int(n), c_int(k), _p(bias), _stream()), "gemm_f32")
        return out
    if k % 8:
        pad = 8 - k % 8
        x2, weight = torch.nn.functional.pad(x2, (0, pad)), torch.nn.functional.pad(weight, (0, pad))
        k += pad
    _check(lib().telb_gemm_f16_f32out(_p(x2), _p(weight), _p(out), c_int(m), c_int(n), c_int(k), _p(bias), c_int(_is_bf16(x)),
                                      _p(Workspace.get(x.device).status), _stream()), "gemm_f16_f32out")
    return out


def stream_norm(stream, weight, eps: float, delta, routed, mult: float, step, offset: float, ids, table, dtype, alpha=None, bias=None,
                table_mult: float = 1.0):
    """See :func:`ops.stream_norm`; ``routed`` carries expert rows (``y``, routing tables ``ws``, weights)."""
    if stream is None:
        t, width, dev = ids.numel(), table.shape[1], table.device
        ids = ids.to(torch.int32).contiguous()
        if table.dtype != dtype:
            raise TypeError(f"stream_norm: embedding table {table.dtype}, activations {dtype}")
    else:
        (t, width), dev = stream.shape, stream.device
        ids = table = None
    for d in (delta, None if routed is None else routed.y):
        if d is not None and d.dtype != dtype:
            raise TypeError(f"stream_norm: update {d.dtype}, activations {dtype}")
    x = torch.empty(t, width, dtype=torch.float32, device=dev)
    h = None if weight is None else torch.empty(t, width, dtype=dtype, device=dev)
    y = ws = w = None
    if routed is not None:
        y, ws, w = routed.y, routed.ws, routed.weights
    code = 2 if dtype == torch.float32 else int(dtype == torch.bfloat16)
    _check(lib().telb_stream_norm(
        _p(ids), _p(table), c_int(table.shape[0] if table is not None else 0), _p(stream), _p(delta.contiguous() if delta is not None else None), _p(y),
        _p(ws.dst_row if ws is not None else None), _p(w), c_int(w.shape[1] if w is not None else 0), c_int(y.shape[1] if y is not None else 0),
        c_float(mult), _p(step), _p(weight), c_float(offset), c_float(eps), _p(alpha), _p(bias), c_float(table_mult), _p(x), _p(h), c_int(t), c_int(width), c_int(code), _stream()), "stream_norm")
    return x, h


class StreamPostParams(ctypes.Structure):
    """Host mirror of ``StreamPostParams`` (``csrc/kernels/stream_post.cu``)."""
    _fields_ = [(n, c_vp) for n in ("ids", "table", "bigram", "last", "x_in", "delta", "weight", "sums", "conv", "history", "out_norm", "x_out", "h", "q_start",
                                    "q_len", "past_len", "slot_ids", "seq_ids")] + \
               [(n, c_ll) for n in ("buckets", "mul_prev", "mul_cur")] + \
               [(n, c_int) for n in ("vocab", "width", "groups", "tokens", "taps", "block_rows", "n_sums", "sum_count")] + [("eps", c_float)]


def _conv_block_rows(tokens: int) -> int:
    """Rows per CTA of the convolution: every block reads the rows in front of it once more, so long steps take longer blocks."""
    return 8 if tokens <= 148 * 8 else 16 if tokens <= 148 * 4 * 16 else 32


def stream_post(stream, delta, weight, groups: int, eps: float, meta: StepMeta, dtype, ids, table, bigram, conv, history, out_norm,
                sums=None):
    """See :func:`ops.stream_post`."""
    f32 = torch.float32
    if dtype not in (torch.bfloat16, f32):
        raise TypeError(f"stream_post: the un-normed stream leaves in bf16 or fp32, not {dtype}")
    if stream is None:
        t, width, dev = ids.numel(), table.shape[1], table.device
        ids = ids.to(torch.int32).contiguous()
        if table.dtype != dtype or (bigram is not None and (bigram.table.dtype != dtype or bigram.table.shape != (bigram.buckets + 1, width))):
            raise TypeError(f"stream_post: embedding tables of {table.dtype}, activations {dtype}")
        if bigram is not None:
            assert bigram.last.dtype == torch.int32 and bigram.last.is_contiguous() and bigram.table.is_contiguous()
    else:
        (t, width), dev = stream.shape, stream.device
        assert stream.dtype == f32 and stream.is_contiguous()
        ids = table = bigram = None
    if delta is not None:
        delta = delta.contiguous()
        assert delta.dtype == dtype and delta.shape == (t, width) and weight.dtype == f32 and weight.numel() == width
    partial, count = sums if sums is not None else (None, 0)
    assert partial is None or (partial.dtype == f32 and partial.is_contiguous() and partial.shape[0] == t and delta is not None)
    taps = 0 if conv is None else conv.shape[0]
    if conv is not None:
        assert conv.dtype == f32 and conv.is_contiguous() and conv.shape[1] == width and out_norm is None
        assert taps == 1 or (history.dtype == f32 and history.is_contiguous() and history.shape[1:] == (taps - 1, width))
    x = torch.empty(t, width, dtype=f32, device=dev)
    h = torch.empty(t, width, dtype=dtype, device=dev)
    ptr = lambda v: None if v is None else _p(v).value
    b = bigram
    p = StreamPostParams(*[ptr(v) for v in (ids, table, None if b is None else b.table, None if b is None else b.last, stream, delta, weight, partial, conv,
                                            history if taps > 1 else None, out_norm, x, h, meta.q_start, meta.q_len, meta.past_len, meta.slot_ids,
                                            meta.seq_ids)],
                         *((0, 0, 0) if b is None else (b.buckets, b.mul_prev, b.mul_cur)), 0 if table is None else table.shape[0], width, groups, t, taps,
                         _conv_block_rows(t), 0 if partial is None else partial.shape[1], count, eps)
    code = 2 if dtype == f32 else 1
    one_row = meta.max_q_len == 1
    _check(lib().telb_stream_post(ctypes.byref(p), c_int(int(one_row)), c_int(code), _stream()), "stream_post", 1 if one_row or not taps else 2)
    return x, h


class StreamSandwichParams(ctypes.Structure):
    """Host mirror of ``StreamSandwichParams`` (``csrc/kernels/stream_sandwich.cu``)."""
    _fields_ = [(n, c_vp) for n in ("ids", "table", "pos_table", "x_in", "y", "e", "dst_row", "topk_w", "post", "norm", "shift", "state", "x_out", "h", "positions",
                                    "q_start", "q_len", "past_len", "slot_ids", "seq_ids")] + \
               [(n, c_int) for n in ("vocab", "max_pos", "width", "tokens", "block_rows", "top_k", "lde")] + [("mult", c_float), ("eps", c_float)]


def _sandwich_block_rows(tokens: int, shifted: bool) -> int:
    """Rows per CTA.  Shifted blocks compute the row in front of them once more, so long steps take longer blocks."""
    if not shifted:
        return 1 if tokens <= 148 * 8 else 2
    return 1 if tokens <= 148 * 2 else 4 if tokens <= 148 * 16 else 8


SANDWICH_WARP_ROWS = (1, 8)      # rows per warp of long steps: as they are, with a shift


def stream_sandwich(stream, eps: float, meta: StepMeta, dtype, ids, table, positions, delta, routed, post, mult: float, norm, shift, state):
    """See :func:`ops.stream_sandwich`; ``routed`` carries expert rows (``y``, routing tables ``ws``, weights)."""
    f32 = torch.float32
    if dtype not in (torch.bfloat16, f32):
        raise TypeError(f"stream_sandwich: rows in bf16 or fp32, not {dtype}")
    if stream is None:
        t, width, dev = ids.numel(), table.shape[1], table.device
        ids = ids.to(torch.int32).contiguous()
    else:
        (t, width), dev = stream.shape, stream.device
        assert stream.dtype == f32 and stream.is_contiguous()
        ids = table = None
    y = ws = w = None
    if routed is not None:
        y, ws, w = routed.y, routed.ws, routed.weights
        assert y.is_contiguous() and y.shape[1] == width and w.shape[0] == t and w.dtype == f32
    if delta is not None:
        delta = delta.contiguous()
        assert delta.shape == (t, width)
    for v in (table, positions, delta, y):
        if v is not None and v.dtype != dtype:
            raise TypeError(f"stream_sandwich: rows of {v.dtype}, activations {dtype}")
    for v in (post, norm, shift):
        assert v is None or (v.dtype == f32 and v.numel() == width and v.is_contiguous())
    assert shift is None or (state.dtype == f32 and state.is_contiguous() and state.shape[1:] == (1, width))
    assert positions is None or (positions.is_contiguous() and positions.shape[1] == width)
    x = torch.empty(t, width, dtype=f32, device=dev)
    h = None if norm is None else torch.empty(t, width, dtype=dtype, device=dev)
    rows = 1 if shift is not None and meta.max_q_len == 1 else _sandwich_block_rows(t, shift is not None)
    p = StreamSandwichParams(*[None if v is None else _p(v).value for v in (
        ids, table, positions, stream, delta, y, None if ws is None else ws.dst_row, w, post, norm, shift, state, x, h, meta.positions, meta.q_start, meta.q_len,
        meta.past_len, meta.slot_ids, meta.seq_ids)], 0 if table is None else table.shape[0], 0 if positions is None else positions.shape[0], width, t, rows,
        0 if w is None else w.shape[1], 0 if y is None else y.shape[1], mult, eps)
    code = 2 if dtype == f32 else 1
    warp_rows = SANDWICH_WARP_ROWS[shift is not None] if t >= 148 * 8 else 0
    _check(lib().telb_stream_sandwich(ctypes.byref(p), c_int(warp_rows), c_int(code), _stream()), "stream_sandwich")
    return x, h


def rope_table(inv_freq: torch.Tensor, attention_factor: float, max_pos: int, device) -> torch.Tensor:
    """``[max_pos, 2 * len(inv_freq)]`` fp32 cos | sin table from fp64 inverse frequencies, built on the device."""
    inv = inv_freq.to(device=device, dtype=torch.float64).contiguous()
    out = torch.empty(max_pos, 2 * inv.numel(), dtype=torch.float32, device=device)
    with torch.cuda.device(out.device):
        _check(lib().telb_rope_table(_p(inv), c_float(float(attention_factor)), _p(out), c_int(max_pos), c_int(inv.numel()), _stream()), "rope_table")
    return out


def mrope_rows(cos_sin: torch.Tensor, positions3: torch.Tensor, sections) -> torch.Tensor:
    """Per-row multimodal RoPE tables ``[T, D]`` gathered from the ordinary table by (temporal, height, width) positions."""
    half = cos_sin.shape[-1] // 2
    if len(sections) != 3 or sum(sections) != half:
        raise ValueError(f"mrope sections {list(sections)} must be three counts summing to {half}")
    cs = cos_sin.float().contiguous()
    p3 = positions3.to(device=cs.device, dtype=torch.int32).contiguous()
    out = torch.empty(p3.shape[1], 2 * half, dtype=torch.float32, device=cs.device)
    _check(lib().telb_mrope_rows(_p(cs), _p(p3), _p(out), c_int(p3.shape[1]), c_int(half), c_int(cs.shape[0]), c_int(int(sections[0])),
                                 c_int(int(sections[1])), _stream()), "mrope_rows")
    return out


def rope_kv_write(qkv, kv_layer, meta: StepMeta, cos_sin, num_q_heads, num_kv_heads, head_dim,
                  q_norm_w=None, k_norm_w=None, eps=1e-6) -> torch.Tensor:
    qkv = qkv.contiguous()
    t = qkv.shape[0]
    q = torch.empty(t, num_q_heads, head_dim, dtype=qkv.dtype, device=qkv.device)
    assert kv_layer.is_contiguous() and kv_layer.dtype == qkv.dtype
    positions = meta.positions
    if meta.rope_rows is not None:          # multimodal RoPE: per-row cos / sin tables prepared by the model
        cos_sin, positions = meta.rope_rows, meta.rope_pos
    _check(lib().telb_rope_kv_write(
        _p(qkv), _p(q), _p(kv_layer), _p(cos_sin), _p(positions), _p(meta.seq_ids), _p(meta.q_start),
        _p(meta.past_len), _p(meta.page_table), _p(meta.kv_offsets), _p(q_norm_w), _p(k_norm_w), c_int(t),
        c_int(num_q_heads), c_int(num_kv_heads), c_int(head_dim), c_int(cos_sin.shape[-1]), c_int(meta.page_size),
        c_int(meta.page_table.shape[1]), c_float(eps), c_int(_dtype_code(qkv)), _stream()), "rope_kv_write")
    return q


_KV_STAGE: Dict[tuple, torch.Tensor] = {}


def kv_fp8_stage(kv_layer: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """The 16-bit staging layer an FP8 KV pool's attention works on (one per device, shape and type, shared by all layers)."""
    key = (kv_layer.device, tuple(kv_layer.shape), dtype)
    st = _KV_STAGE.get(key)
    if st is None:
        st = _KV_STAGE[key] = torch.zeros(kv_layer.shape, dtype=dtype, device=kv_layer.device)
    return st


def kv_fp8_load(kv_layer: torch.Tensor, stage: torch.Tensor, meta: StepMeta, scales: torch.Tensor, window: int = 0) -> None:
    """Expand the pages that hold the step's cached tokens from the FP8 layer ``[pages, 2, Hkv, P, D]`` into ``stage``."""
    _, _, hkv, psz, d = kv_layer.shape
    _check(lib().telb_kv_fp8_load(_p(kv_layer), _p(stage), _p(meta.past_len), _p(meta.page_table), _p(scales), c_int(meta.num_seqs),
                                  c_int(meta.page_table.shape[1]), c_int(psz), c_int(hkv), c_int(d), c_int(window or 0),
                                  c_int(_is_bf16(stage)), _stream()), "kv_fp8_load")


def kv_fp8_store(kv_layer: torch.Tensor, stage: torch.Tensor, meta: StepMeta, scales: torch.Tensor, q: Optional[torch.Tensor] = None):
    """Quantise the step's new K / V rows from ``stage`` into the FP8 layer and write the rounded values back to ``stage``.
    With ``q`` ``[T, Hq, D]`` the same launch also casts the query rows to E4M3 and returns them (else None)."""
    _, _, hkv, psz, d = kv_layer.shape
    q8 = None
    if q is not None:
        q = q.contiguous()
        q8 = torch.empty(q.shape, dtype=torch.float8_e4m3fn, device=q.device)
    _check(lib().telb_kv_fp8_store(_p(kv_layer), _p(stage), _p(meta.seq_ids), _p(meta.q_start), _p(meta.past_len), _p(meta.page_table),
                                   _p(meta.kv_offsets), _p(scales), c_int(meta.num_tokens), c_int(meta.page_table.shape[1]), c_int(psz),
                                   c_int(hkv), c_int(d), c_int(_is_bf16(stage)), _p(q), _p(q8), c_int(q.shape[1] if q is not None else 0),
                                   _stream()), "kv_fp8_store")
    return q8


def fp8_decode_ok(q_shape, hkv: int, meta: StepMeta) -> bool:
    """Whether the decode kernel that reads FP8 pages in place covers this step (decode-shaped, head_dim 128)."""
    t, hq, d = q_shape
    group = hq // hkv
    return (meta.tree_mask is None and d == 128 and meta.max_q_len * group <= 16 and 16 % group == 0
            and os.environ.get("TELB_DISABLE_FP8_DECODE_ATTN", "0") != "1")


def paged_attention_decode_fp8(q8: torch.Tensor, kv_layer: torch.Tensor, meta: StepMeta, scale: float, sliding_window, kv_scales: torch.Tensor,
                               out_dtype: torch.dtype, out_scale: Optional[torch.Tensor] = None, sinks: Optional[torch.Tensor] = None,
                               splits: Optional[int] = None):
    """Decode-shaped attention over FP8 (E4M3) pages read in place.  ``q8``: the query rows cast to E4M3.  Returns 16-bit rows
    ``[T, Hq, D]`` of ``out_dtype``, or ``QuantActs`` over ``[T, Hq * D]`` when ``out_scale`` (the next projection's NVFP4 input
    scale) is given."""
    t, hq, d = q8.shape
    hkv = kv_layer.shape[2]
    if splits is None:
        splits = _decode_splits(meta, hkv)
    ws = Workspace.get(q8.device)
    L = lib()
    out = xq = sf = None
    if out_scale is None:
        out = torch.empty(t, hq, d, dtype=out_dtype, device=q8.device)
    else:
        L.telb_nvfp4_sf_bytes.restype = c_ll
        xq = torch.empty(t, hq * d // 2, dtype=torch.uint8, device=q8.device)
        sf = _sf_buffer(L.telb_nvfp4_sf_bytes(c_ll(t), c_int(hq * d)), hq * d, q8.device)
    if sinks is not None:
        sinks = sinks.to(device=q8.device, dtype=torch.float32).contiguous()
    _check(L.telb_paged_attention_decode_fp8(
        _p(q8), _p(kv_layer), _p(out), _p(xq), _p(sf), _p(out_scale), _p(kv_scales), _p(meta.q_start), _p(meta.q_len), _p(meta.past_len),
        _p(meta.page_table), c_int(meta.num_seqs), c_int(t), c_int(meta.max_q_len), c_int(kv_layer.shape[0]), c_int(meta.page_table.shape[1]),
        c_int(meta.page_size), c_int(hq), c_int(hkv), c_int(d), c_float(scale), c_int(sliding_window or 0), c_int(splits), _p(ws.attn_ws),
        c_ll(ws.attn_ws.numel()), c_int(1 if out_dtype == torch.bfloat16 else 0), _p(ws.status), _p(sinks), _stream()),
        "paged_attention_decode_fp8", 2 if splits > 1 else 1)
    return out if out_scale is None else QuantActs(xq, sf, (t, hq * d), out_dtype)


def _visible_len(meta: StepMeta, chunk: int, window: int = 0) -> int:
    """Most keys that rows of one tile of the step can see."""
    n = min(meta.max_seq_len, chunk) if chunk > 0 else meta.max_seq_len
    return min(n, window + 128) if window > 0 else n


def _attn_splits(meta: StepMeta, hkv: int, group: int, chunk: int = 0, window: int = 0) -> int:
    tq = 128 // group
    qtiles = (meta.max_q_len + tq - 1) // tq
    ctas = meta.num_seqs * hkv * qtiles
    if ctas >= 148 or meta.max_q_len > 4 * tq:
        return 1
    kv_tiles = max(1, (_visible_len(meta, chunk, window) + 63) // 64)
    return max(1, min((2 * 148 + ctas - 1) // ctas, kv_tiles, 32))


def _decode_splits(meta: StepMeta, hkv: int, chunk: int = 0, window: int = 0) -> int:
    ctas = meta.num_seqs * hkv
    if ctas >= 148:
        return 1
    tiles = max(1, (_visible_len(meta, chunk, window) + 127) // 128)
    return max(1, min((148 + ctas - 1) // ctas, tiles, 32))


def paged_attention(q, kv_layer, meta: StepMeta, scale, sliding_window=None, sinks=None, splits: Optional[int] = None,
                    kernel: Optional[str] = None, trace: Optional[torch.Tensor] = None, causal: bool = True,
                    skip_thr: Optional[torch.Tensor] = None, skip_stats: Optional[torch.Tensor] = None, chunk: int = 0,
                    fp32_weights: bool = False, back: Optional[tuple] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Paged GQA attention.  Decode-shaped steps (``max_q_len * Hq/Hkv <= 16``, head_dim 128, causal)
    run the token-major XQA-style kernel; everything else the row-major tile kernel.
    ``kernel`` forces ``"decode"`` or ``"tile"``; ``causal=False`` lets every row see every token of its sequence; ``chunk`` > 0 limits
    a row to the keys of its own ``chunk``-token block; ``fp32_weights`` feeds the probabilities to the 16-bit P·V product as high + low
    halves.  fp32 rows and head sizes without a tensor-core form run on the CUDA cores."""
    if not causal:
        sliding_window, kernel = -1, "tile"
    if sinks is not None:
        sinks = sinks.to(device=q.device, dtype=torch.float32).contiguous()
    q = q.contiguous()
    t, hq, d = q.shape
    hkv = kv_layer.shape[2]
    group = hq // hkv
    table, mult = back if back is not None else (None, 1.0)
    if out is None:
        out = torch.empty_like(q)
        ld_out = hq * d
    else:                                   # rows of a wider buffer
        assert out.shape == (t, hq * d) and out.dtype == q.dtype and out.stride(1) == 1 and out.stride(0) % 8 == 0 and (back is not None or out.is_contiguous())
        ld_out = out.stride(0)
    if back is not None and (table.dtype != torch.float32 or not table.is_contiguous() or table.shape[1] != d or meta.tree_mask is not None):
        raise ValueError("rotated values: an fp32 table row per position and causal steps")
    win = sliding_window if sliding_window and sliding_window > 0 else 0
    tm = meta.tree_mask
    if q.dtype == torch.float32 or d not in (64, 128, 256):
        if tm is not None or not causal or skip_thr is not None or meta.skip_thr is not None:
            raise ValueError("fp32 / odd-sized attention covers causal, windowed and chunked masks only")
        _check(lib().telb_paged_attention_simt(
            _p(q), _p(kv_layer), _p(out), _p(meta.q_start), _p(meta.past_len), _p(meta.seq_ids), _p(meta.page_table), c_int(t),
            c_int(meta.page_table.shape[1]), c_int(meta.page_size), c_int(hq), c_int(hkv), c_int(d), c_float(scale), c_int(sliding_window or 0),
            c_int(chunk), _p(sinks), _p(table), c_float(mult), c_ll(ld_out), c_int(_dtype_code(q)), _stream()), "paged_attention_simt")
        return out
    ws = Workspace.get(q.device)
    decode_ok = (tm is None and d == 128 and meta.max_q_len * group <= 16 and 16 % group == 0)
    if skip_thr is None:
        skip_thr = meta.skip_thr            # per-sequence skip-softmax thresholds of the step (prefill-size steps only)
    if skip_thr is not None:
        skip_thr = skip_thr.to(device=q.device, dtype=torch.float32).contiguous()
        if kernel is None and meta.max_q_len * group > 16:
            kernel = "tile"
    use_decode = decode_ok if kernel is None else (kernel == "decode")
    if use_decode:
        if not decode_ok:
            raise ValueError("step is not decode-shaped")
        if splits is None:
            splits = _decode_splits(meta, hkv, chunk, win)
        _check(lib().telb_paged_attention_decode_traced(
            _p(q), _p(kv_layer), _p(out), _p(meta.q_start), _p(meta.q_len), _p(meta.past_len), _p(meta.page_table),
            c_int(meta.num_seqs), c_int(t), c_int(meta.max_q_len), c_int(kv_layer.shape[0]), c_int(meta.page_table.shape[1]),
            c_int(meta.page_size), c_int(hq), c_int(hkv), c_int(d), c_float(scale), c_int(sliding_window or 0), c_int(splits),
            _p(ws.attn_ws), c_ll(ws.attn_ws.numel()), c_int(_is_bf16(q)), _p(ws.status), _p(trace), _p(sinks), c_int(chunk), c_int(int(fp32_weights)),
            _p(table), c_float(mult), _p(meta.positions), c_ll(ld_out), _stream()),
            "paged_attention_decode", 2 if splits > 1 else 1)
        return out
    if splits is None:
        splits = _attn_splits(meta, hkv, group, chunk, win)
    _check(lib().telb_paged_attention(
        _p(q), _p(kv_layer), _p(out), _p(meta.q_start), _p(meta.q_len), _p(meta.past_len), _p(meta.page_table),
        _p(tm), c_int(tm.shape[1] if tm is not None else 0), c_int(meta.num_seqs), c_int(t), c_int(meta.max_q_len),
        c_int(kv_layer.shape[0]), c_int(meta.page_table.shape[1]), c_int(meta.page_size), c_int(hq), c_int(hkv),
        c_int(d), c_float(scale), c_int(sliding_window or 0), c_int(splits), _p(ws.attn_ws), c_ll(ws.attn_ws.numel()),
        c_int(_is_bf16(q)), _p(ws.status), _p(sinks), _p(skip_thr), _p(skip_stats), c_int(chunk), c_int(int(fp32_weights)),
        _p(table), c_float(mult), _p(meta.positions), c_ll(ld_out), _stream()), "paged_attention", 2 if splits > 1 else 1)
    return out


def decode_attention_quant_ok(q_shape, hkv: int, meta: StepMeta) -> bool:
    """Whether :func:`paged_attention_quant` covers this step (the decode-shaped kernel, head_dim 128)."""
    t, hq, d = q_shape
    group = hq // hkv
    return (meta.tree_mask is None and d == 128 and meta.max_q_len * group <= 16 and 16 % group == 0
            and os.environ.get("TELB_DISABLE_ATTN_QUANT_FUSION", "0") != "1")


def paged_attention_quant(q, kv_layer, meta: StepMeta, scale, sliding_window, out_scale: torch.Tensor,
                          splits: Optional[int] = None, sinks: Optional[torch.Tensor] = None) -> "QuantActs":
    """Decode-shaped paged attention whose epilogue (or split merge) writes NVFP4 rows ``[T, Hq * D]`` quantised with the
    global scale ``out_scale`` of the projection that follows, instead of 16-bit rows and a quantisation kernel."""
    q = q.contiguous()
    t, hq, d = q.shape
    hkv = kv_layer.shape[2]
    if not decode_attention_quant_ok(q.shape, hkv, meta):
        raise ValueError("step is not decode-shaped")
    if splits is None:
        splits = _decode_splits(meta, hkv)
    L = lib()
    L.telb_nvfp4_sf_bytes.restype = c_ll
    width = hq * d
    xq = torch.empty(t, width // 2, dtype=torch.uint8, device=q.device)
    sf = _sf_buffer(L.telb_nvfp4_sf_bytes(c_ll(t), c_int(width)), width, q.device)
    ws = Workspace.get(q.device)
    _check(L.telb_paged_attention_decode_quant(
        _p(q), _p(kv_layer), _p(xq), _p(sf), _p(out_scale), _p(meta.q_start), _p(meta.q_len), _p(meta.past_len), _p(meta.page_table),
        c_int(meta.num_seqs), c_int(t), c_int(meta.max_q_len), c_int(kv_layer.shape[0]), c_int(meta.page_table.shape[1]),
        c_int(meta.page_size), c_int(hq), c_int(hkv), c_int(d), c_float(scale), c_int(sliding_window or 0), c_int(splits),
        _p(ws.attn_ws), c_ll(ws.attn_ws.numel()), c_int(_is_bf16(q)), _p(ws.status),
        _p(None if sinks is None else sinks.to(device=q.device, dtype=torch.float32).contiguous()), _stream()),
        "paged_attention_decode_quant", 2 if splits > 1 else 1)
    return QuantActs(xq, sf, (t, width), q.dtype)


def argmax(logits: torch.Tensor) -> torch.Tensor:
    assert logits.dim() == 2 and logits.stride(1) == 1
    out = torch.empty(logits.shape[0], dtype=torch.int32, device=logits.device)
    dt = 2 if logits.dtype == torch.float32 else _is_bf16(logits)
    ws = Workspace.get(logits.device)
    _check(lib().telb_argmax(_p(logits), _p(out), c_ll(logits.shape[0]), c_int(logits.shape[1]),
                             c_ll(logits.stride(0)), c_int(dt), _p(ws.argmax_keys), _p(ws.argmax_counters),
                             c_int(ws.argmax_keys.numel()), _stream()), "argmax")
    return out




# ---- NVFP4 -----------------------------------------------------------------------------------


def nvfp4_swizzle_scales(weight_scale: torch.Tensor) -> torch.Tensor:
    """Row-major E4M3 block scales ``[rows, K/16]`` → the 512-byte atom layout the tensor core reads
    (``[ceil(rows/128), K/64 padded to whole 256-element stages, 512]`` bytes)."""
    sf = weight_scale.view(torch.uint8).contiguous()
    rows, kb = sf.shape
    k = kb * 16
    L = lib()
    L.telb_nvfp4_sf_bytes.restype = c_ll
    nbytes = L.telb_nvfp4_sf_bytes(c_ll(rows), c_int(k))
    out = torch.empty(nbytes, dtype=torch.uint8, device=sf.device)
    _check(L.telb_nvfp4_swizzle_scales(_p(sf), _p(out), c_ll(rows), c_int(k), _stream()), "nvfp4_swizzle_scales")
    return out


class QuantActs:
    """Activations already quantised to NVFP4 by their producer (packed codes + atom-layout scales)."""

    __slots__ = ("xq", "sf", "shape", "dtype", "ag_wait")

    def __init__(self, xq: torch.Tensor, sf: torch.Tensor, shape, dtype):
        self.xq, self.sf, self.shape, self.dtype = xq, sf, tuple(shape), dtype
        self.ag_wait = None      # GemmFusion when the rows are still being gathered from peers

    @property
    def is_cuda(self) -> bool:
        return True


def _sf_buffer(nbytes: int, k: int, device) -> torch.Tensor:
    # Rows beyond M only feed accumulator rows that are never stored, so they may hold anything;
    # K padding multiplies real rows and must be zero.
    return (torch.zeros if k % 256 else torch.empty)(nbytes, dtype=torch.uint8, device=device)


def rmsnorm_quant(x: torch.Tensor, residual: Optional[torch.Tensor], weight: torch.Tensor, eps: float,
                  global_scale: torch.Tensor):
    """``(residual add +) RMSNorm`` whose output is written as NVFP4 only.  Returns
    ``(QuantActs, new_residual)`` (``new_residual`` is ``x`` itself when there is no residual)."""
    x = x.contiguous()
    m, k = x.shape
    L = lib()
    L.telb_nvfp4_sf_bytes.restype = c_ll
    nbytes = L.telb_nvfp4_sf_bytes(c_ll(m), c_int(k))
    xq = torch.empty(m, k // 2, dtype=torch.uint8, device=x.device)
    sf = _sf_buffer(nbytes, k, x.device)
    res_out = torch.empty_like(x) if residual is not None else None
    _check(L.telb_rmsnorm_quant(_p(x), _p(residual), _p(weight), _p(res_out), c_vp(0), _p(xq), _p(sf), _p(global_scale),
                                c_ll(m), c_int(k), c_float(eps), c_int(_is_bf16(x)), _stream()), "rmsnorm_quant")
    return QuantActs(xq, sf, (m, k), x.dtype), (res_out if residual is not None else x)


def gemm_nvfp4_swiglu(x: "QuantActs", weight: torch.Tensor, w_sf: torch.Tensor, alpha: torch.Tensor, out_scale: torch.Tensor,
                      fusion=None) -> "QuantActs":
    """Gate/up projection whose epilogue applies SwiGLU and quantises to NVFP4: ``weight [2·I, K/2]`` holds blocks of 64
    gate rows alternating with their up rows; returns the quantised ``[M, I]`` activations (M > 128)."""
    m, n, k = x.xq.shape[0], weight.shape[0], x.xq.shape[1] * 2
    inter = n // 2
    L = lib()
    L.telb_nvfp4_sf_bytes.restype = c_ll
    xq = torch.empty(m, inter // 2, dtype=torch.uint8, device=weight.device)
    sf = _sf_buffer(L.telb_nvfp4_sf_bytes(c_ll(m), c_int(inter)), inter, weight.device)
    ws = Workspace.get(weight.device)
    _check(L.telb_gemm_nvfp4_swiglu(_p(x.xq), _p(x.sf), _p(weight), _p(w_sf), _p(alpha), _p(xq), _p(sf), _p(out_scale), c_int(m), c_int(n),
                                    c_int(k), c_int(1 if x.dtype == torch.bfloat16 else 0), _p(ws.status),
                                    ctypes.byref(fusion) if fusion is not None else c_vp(0), _stream()), "gemm_nvfp4_swiglu")
    return QuantActs(xq, sf, (m, inter), x.dtype)


def gemm_skinny_swiglu(x: "QuantActs", weight: torch.Tensor, w_sf: torch.Tensor, alpha: torch.Tensor, out_scale: torch.Tensor,
                       fusion=None) -> "QuantActs":
    """Decode-size form of :func:`gemm_nvfp4_swiglu` (M <= 64): the swapped-operand, cluster split-K kernel applies SwiGLU and
    quantises in its epilogue, so a decode step has no separate activation kernel between the gate/up and down projections."""
    m, n, k = x.xq.shape[0], weight.shape[0], x.xq.shape[1] * 2
    inter = n // 2
    L = lib()
    L.telb_nvfp4_sf_bytes.restype = c_ll
    xq = torch.empty(m, inter // 2, dtype=torch.uint8, device=weight.device)
    sf = _sf_buffer(L.telb_nvfp4_sf_bytes(c_ll(m), c_int(inter)), inter, weight.device)
    ws = Workspace.get(weight.device)
    _check(L.telb_gemm_skinny_swiglu(c_int(1), _p(x.xq), _p(x.sf), _p(weight), _p(w_sf), _p(alpha), _p(xq), _p(sf), _p(out_scale), c_int(m),
                                     c_int(n), c_int(k), c_int(1 if x.dtype == torch.bfloat16 else 0), _p(ws.status),
                                     ctypes.byref(fusion) if fusion is not None else c_vp(0), _stream()), "gemm_skinny_swiglu")
    return QuantActs(xq, sf, (m, inter), x.dtype)


def swiglu_quant(gate_up: torch.Tensor, global_scale: torch.Tensor, interleaved: bool = False, moe_ws=None) -> QuantActs:
    """``moe_ws``: the routing tables of a grouped (mixture-of-experts) buffer; its padding rows are skipped."""
    gate_up = gate_up.contiguous()
    m = gate_up.shape[0]
    inter = gate_up.shape[1] // 2
    L = lib()
    L.telb_nvfp4_sf_bytes.restype = c_ll
    nbytes = L.telb_nvfp4_sf_bytes(c_ll(m), c_int(inter))
    xq = torch.empty(m, inter // 2, dtype=torch.uint8, device=gate_up.device)
    sf = _sf_buffer(nbytes, inter, gate_up.device)
    tile_rows = c_vp(moe_ws.tile_expert.data_ptr() + 4 * moe_ws.max_tiles) if moe_ws is not None else c_vp(0)
    _check(L.telb_swiglu_quant_rows(_p(gate_up), _p(xq), _p(sf), _p(global_scale), c_ll(m), c_int(inter),
                                    c_int(_is_bf16(gate_up)), c_int(1 if interleaved else 0), tile_rows, _stream()), "swiglu_quant")
    return QuantActs(xq, sf, (m, inter), gate_up.dtype)


def nvfp4_quantize(x: torch.Tensor, global_scale: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """Quantise activations ``[M,K]`` to packed E2M1 ``[M,K/2]`` + atom-layout E4M3 scales."""
    x = x.contiguous()
    m, k = x.shape
    L = lib()
    L.telb_nvfp4_sf_bytes.restype = c_ll
    nbytes = L.telb_nvfp4_sf_bytes(c_ll(m), c_int(k))
    xq = torch.empty(m, k // 2, dtype=torch.uint8, device=x.device)
    sf = _sf_buffer(nbytes, k, x.device)
    _check(L.telb_nvfp4_quantize(_p(x), _p(xq), _p(sf), _p(global_scale), c_ll(m), c_int(k), c_int(_is_bf16(x)), _stream()),
           "nvfp4_quantize")
    return xq, sf


def gemm_nvfp4(xq, x_sf, wq, w_sf, alpha, out_dtype, bias=None, residual=None, mode: int = 0, splits: int = 0):
    m, n, k = xq.shape[0], wq.shape[0], xq.shape[1] * 2
    out = torch.empty(m, n, dtype=out_dtype, device=xq.device)
    ws = Workspace.get(xq.device)
    _check(lib().telb_gemm_nvfp4(_p(xq), _p(x_sf), _p(wq), _p(w_sf), _p(out), c_int(m), c_int(n), c_int(k), _p(alpha),
                                 _p(bias), _p(residual), c_int(1 if out_dtype == torch.bfloat16 else 0), _p(ws.gemm_ws),
                                 c_ll(ws.gemm_ws.numel()), _p(ws.counters), c_int(ws.counters.numel()), _p(ws.status),
                                 c_int(mode), c_int(splits), _stream()), "gemm_nvfp4")
    return out


def nvfp4_linear(x, weight, weight_sf_atoms, alpha, input_scale, bias=None, quantize_activations=True):
    """NVFP4 linear: dynamic per-16 activation quantisation (calibrated global scale) + block-scaled GEMM."""
    if not quantize_activations:
        raise NotImplementedError("W4A16 NVFP4 runs through the W4A4 tensor-core path only when activations are quantised")
    if isinstance(x, QuantActs):
        return gemm_nvfp4(x.xq, x.sf, weight, weight_sf_atoms, alpha, x.dtype, bias)
    lead = x.shape[:-1]
    x2 = x.reshape(-1, x.shape[-1])
    xq, x_sf = nvfp4_quantize(x2, input_scale)
    out = gemm_nvfp4(xq, x_sf, weight, weight_sf_atoms, alpha, x.dtype, bias)
    return out.reshape(*lead, weight.shape[0])


class GemmFusion(ctypes.Structure):
    """Host mirror of ``TelbGemmFusion`` (``csrc/kernels/gemm_common.cuh``)."""
    _fields_ = [("rs_out", c_vp * 8), ("rs_world", c_int), ("rs_rank", c_int), ("rs_rows_per_rank", c_int), ("pad0", c_int),
                ("ag_flags", c_vp), ("ag_epoch", c_vp), ("ag_world", c_int), ("ag_rows_per_rank", c_int)]


def gemm_fused(x, weight, fusion: GemmFusion, *, w_sf=None, alpha=None, bias=None, out=None, out_dtype=None):
    """Large-M GEMM with a fused tensor-parallel collective: ``x`` is 16-bit ``[M, K]`` or ``QuantActs``.
    With a reduce-scatter epilogue the rows land in the peers' partial buffers and nothing is returned."""
    ws = Workspace.get(weight.device)
    scatter = fusion.rs_world > 1
    if isinstance(x, QuantActs):
        m, n, k = x.xq.shape[0], weight.shape[0], x.xq.shape[1] * 2
        dt = out_dtype or x.dtype
        if out is None and not scatter:
            out = torch.empty(m, n, dtype=dt, device=weight.device)
        _check(lib().telb_gemm_nvfp4_fused(_p(x.xq), _p(x.sf), _p(weight), _p(w_sf), _p(out), c_int(m), c_int(n), c_int(k), _p(alpha),
                                           _p(bias), c_int(1 if dt == torch.bfloat16 else 0), _p(ws.status), ctypes.byref(fusion),
                                           _stream()), "gemm_nvfp4_fused")
        return out
    m, k = x.shape
    n = weight.shape[0]
    if out is None and not scatter:
        out = torch.empty(m, n, dtype=x.dtype, device=x.device)
    _check(lib().telb_gemm_f16_fused(_p(x), _p(weight), _p(out), c_int(m), c_int(n), c_int(k), _p(bias), _p(alpha), c_int(_is_bf16(x)),
                                     _p(ws.status), ctypes.byref(fusion), _stream()), "gemm_f16_fused")
    return out


def gemm_skinny(x, weight, *, x_sf=None, w_sf=None, alpha=None, bias=None, residual=None, out_dtype=None, ranks: int = 0):
    """Decode-size GEMM (M <= 128) with an explicit cluster size (``ranks`` K-slices; 0 = choose).
    16-bit operands when no scale tensors are given, NVFP4 otherwise."""
    kind = 1 if w_sf is not None else 0
    m = x.shape[0]
    n = weight.shape[0]
    k = x.shape[1] * (2 if kind else 1)
    dt = out_dtype or x.dtype
    out = torch.empty(m, n, dtype=dt, device=x.device)
    ws = Workspace.get(x.device)
    _check(lib().telb_gemm_skinny(c_int(kind), _p(x), _p(x_sf), _p(weight), _p(w_sf), _p(out), c_int(m), c_int(n), c_int(k),
                                  _p(alpha), _p(bias), _p(residual), c_int(1 if dt == torch.bfloat16 else 0), _p(ws.status),
                                  c_int(ranks), _stream()), "gemm_skinny")
    return out


INT4_GEMV_MAX_ROWS = 0 if os.environ.get("TELB_DISABLE_INT4_GEMV", "0") == "1" else 4


def gemm_int4_awq(x: torch.Tensor, wq: torch.Tensor, scales: torch.Tensor, group: int, bias=None, residual=None, ranks: int = 0):
    """W4A16 linear on ModelOpt-prepacked INT4 weights (``wq [N/2, K]`` uint8, ``scales [N, K/group]`` in ``x``'s dtype).
    Decode-size steps (M <= 128) expand the 4-bit tiles inside the GEMM kernel, so only 4-bit weights cross HBM; larger
    steps expand the matrix once into a temporary and run the dense tensor-core GEMM (compute-bound there)."""
    lead = x.shape[:-1]
    x2 = x.reshape(-1, x.shape[-1])
    if not x2.is_contiguous():
        x2 = x2.contiguous()
    m, k = x2.shape
    n = wq.shape[0] * 2
    if scales.dtype != x.dtype:
        scales = scales.to(x.dtype)
    ok = n % 2 == 0 and k % 64 == 0 and group >= 64 and group % 64 == 0 and k % group == 0
    if m <= INT4_GEMV_MAX_ROWS and ok and m * k * 2 <= 200 * 1024:
        # one to four rows: a CUDA-core GEMV streams the packed weights once (the tensor-core tile would be almost empty)
        out = torch.empty(m, n, dtype=x.dtype, device=x.device)
        _check(lib().telb_gemv_int4(_p(x2), _p(wq), _p(scales.contiguous()), _p(out), c_int(m), c_int(n), c_int(k), c_int(group), _p(bias),
                                    _p(residual.reshape(m, n).contiguous() if residual is not None else None), c_int(_is_bf16(x)), _stream()),
               "gemv_int4")
        return out.reshape(*lead, n)
    if m <= 128 and ok:
        out = torch.empty(m, n, dtype=x.dtype, device=x.device)
        ws = Workspace.get(x.device)
        _check(lib().telb_gemm_skinny_int4(_p(x2), _p(wq), _p(scales.contiguous()), _p(out), c_int(m), c_int(n), c_int(k), c_int(group), _p(bias),
                                           _p(residual), c_int(_is_bf16(x)), _p(ws.status), c_int(ranks), _stream()), "gemm_skinny_int4")
        return out.reshape(*lead, n)
    dense = torch.empty(n, k, dtype=x.dtype, device=x.device)
    _check(lib().telb_int4_awq_expand(_p(wq), _p(scales.contiguous()), _p(dense), c_int(n), c_int(k), c_int(group), c_int(_is_bf16(x)), _stream()),
           "int4_awq_expand")
    return gemm(x2, dense, bias=bias, residual=residual).reshape(*lead, n)


# ---- sampling ----------------------------------------------------------------------------------


def _logit_dtype(t: torch.Tensor) -> int:
    return 2 if t.dtype == torch.float32 else _is_bf16(t)


def sample(logits, temperature, top_k, top_p, uniforms) -> torch.Tensor:
    assert logits.dim() == 2 and logits.stride(1) == 1
    rows, vocab = logits.shape
    out = torch.empty(rows, dtype=torch.int32, device=logits.device)
    _check(lib().telb_sample(_p(logits), c_ll(logits.stride(0)), c_int(rows), c_int(vocab),
                             _p(temperature.to(torch.float32).contiguous()), _p(top_k.to(torch.int32).contiguous()),
                             _p(top_p.to(torch.float32).contiguous()), _p(uniforms.to(torch.float32).contiguous()), _p(out),
                             c_int(_logit_dtype(logits)), _stream()), "sample")
    return out


def token_logprobs(logits, tokens, k: int):
    """``(chosen [rows] fp32, top_ids [rows, k] int32, top_values [rows, k] fp32)``: log-probability of ``tokens[row]`` and the ``k``
    most likely tokens of every row under ``softmax(logits[row])``."""
    assert logits.dim() == 2 and logits.stride(1) == 1 and 0 <= k <= 32
    rows, vocab = logits.shape
    tok = tokens.to(device=logits.device, dtype=torch.int32).contiguous()
    chosen = torch.empty(rows, dtype=torch.float32, device=logits.device)
    ids = torch.empty(rows, max(k, 1), dtype=torch.int32, device=logits.device)
    vals = torch.empty(rows, max(k, 1), dtype=torch.float32, device=logits.device)
    _check(lib().telb_token_logprobs(_p(logits), c_ll(logits.stride(0)), c_int(rows), c_int(vocab), _p(tok), c_int(k), _p(chosen), _p(ids),
                                     _p(vals), c_int(_logit_dtype(logits)), _stream()), "token_logprobs")
    return chosen, ids[:, :k], vals[:, :k]


def apply_token_bitmask(logits: torch.Tensor, bitmask: torch.Tensor) -> torch.Tensor:
    """In place: entries whose bit is 0 in ``bitmask [rows, ceil(V/32)]`` become very negative."""
    _check(lib().telb_apply_token_bitmask(_p(logits), c_ll(logits.stride(0)), c_int(logits.shape[0]), c_int(logits.shape[1]),
                                          _p(bitmask.to(torch.int32).contiguous()), c_int(_logit_dtype(logits)), _stream()),
           "apply_token_bitmask")
    return logits


# ---- mixture of experts -------------------------------------------------------------------------


def moe_route_softmax_topk(logits, top_k, renormalize=True, bias=None, sigmoid=False, n_group=1, topk_group=1,
                           scaling=1.0):
    logits = logits.contiguous()
    t, e = logits.shape
    w = torch.empty(t, top_k, dtype=torch.float32, device=logits.device)
    idx = torch.empty(t, top_k, dtype=torch.int32, device=logits.device)
    _check(lib().telb_moe_route(_p(logits), _p(w), _p(idx), _p(bias.float().contiguous() if bias is not None else None), c_int(t), c_int(e), c_int(top_k), c_int(int(renormalize)),
                                c_int(int(sigmoid)), c_int(n_group), c_int(topk_group), c_float(scaling), c_int(_logit_dtype(logits)),
                                _stream()), "moe_route")
    return w, idx


def moe_route_chosen(logits: torch.Tensor, top_k: int):
    """Top-k of fp32 logits (rows may be a column slice of a wider tensor) and the softmax over the chosen ones."""
    if logits.dtype != torch.float32 or logits.stride(1) != 1:
        raise TypeError("moe_route_chosen takes fp32 rows")
    t, e = logits.shape
    w = torch.empty(t, top_k, dtype=torch.float32, device=logits.device)
    idx = torch.empty(t, top_k, dtype=torch.int32, device=logits.device)
    _check(lib().telb_moe_route_chosen(_p(logits), c_int(logits.stride(0)), _p(w), _p(idx), c_int(t), c_int(e), c_int(top_k), _stream()),
           "moe_route_chosen")
    return w, idx


def clamped_glu(gate_up: torch.Tensor, limit: float, alpha: float, ws: Optional["MoeWorkspace"] = None, up_offset: float = 1.0) -> torch.Tensor:
    """``g σ(alpha g) (u + up_offset)`` over ``[gate | up]`` rows, both clamped unless ``limit`` is 0; with ``ws`` the rows of the padded expert
    layout that hold no token are skipped."""
    rows, two = gate_up.shape
    out = torch.empty(rows, two // 2, dtype=gate_up.dtype, device=gate_up.device)
    tile_rows = c_vp(ws.tile_expert.data_ptr() + 4 * ws.max_tiles) if ws is not None else c_vp(0)
    _check(lib().telb_clamped_glu(_p(gate_up), _p(out), tile_rows, c_int(rows), c_int(two // 2), c_float(limit), c_float(alpha), c_float(up_offset),
                                  c_int(_dtype_code(gate_up)), _stream()), "clamped_glu")
    return out


class MoeWorkspace:
    """Routing tables of one MoE call over the padded row space (every expert segment is a multiple
    of 128 rows, so a 128-row tile belongs to exactly one expert)."""

    def __init__(self, tokens: int, top_k: int, experts_local: int, device):
        slots = tokens * top_k
        self.max_tiles = (slots + 127) // 128 + experts_local
        self.rows_pad = self.max_tiles * 128
        self.dst_row = torch.empty(slots, dtype=torch.int32, device=device)
        # [0, max_tiles): expert of each 128-row tile (-1 = unused); [max_tiles, 2 max_tiles): rows in use in each tile
        self.tile_expert = torch.empty(2 * self.max_tiles, dtype=torch.int32, device=device)
        self.counts = torch.empty(1, dtype=torch.int32, device=device)


def moe_align(topk_idx: torch.Tensor, experts: int, expert_lo: int, expert_hi: int) -> MoeWorkspace:
    t, k = topk_idx.shape
    ws = MoeWorkspace(t, k, expert_hi - expert_lo, topk_idx.device)
    _check(lib().telb_moe_align(_p(topk_idx), _p(ws.dst_row), _p(ws.tile_expert), _p(ws.counts), c_int(t * k), c_int(experts),
                                c_int(expert_lo), c_int(expert_hi), c_int(ws.max_tiles), _stream()), "moe_align")
    return ws


def moe_gather(x: torch.Tensor, ws: MoeWorkspace, top_k: int, quant_scale: Optional[torch.Tensor]):
    """Routed rows in expert order: NVFP4 ``QuantActs`` when ``quant_scale`` is given, else 16-bit."""
    x = x.contiguous()
    t, h = x.shape
    if quant_scale is None:
        out = torch.empty(ws.rows_pad, h, dtype=x.dtype, device=x.device)
        # a plain copy: an fp32 row travels as twice as many 16-bit elements
        _check(lib().telb_moe_gather(_p(x), _p(ws.dst_row), _p(out), c_vp(0), c_vp(0), c_vp(0), c_int(t * top_k), c_int(top_k),
                                     c_int(h * x.element_size() // 2), c_int(1), _stream()), "moe_gather")
        return out
    L = lib()
    L.telb_nvfp4_sf_bytes.restype = c_ll
    xq = torch.empty(ws.rows_pad, h // 2, dtype=torch.uint8, device=x.device)
    sf = _sf_buffer(L.telb_nvfp4_sf_bytes(c_ll(ws.rows_pad), c_int(h)), h, x.device)
    _check(L.telb_moe_gather(_p(x), _p(ws.dst_row), c_vp(0), _p(xq), _p(sf), _p(quant_scale), c_int(t * top_k), c_int(top_k),
                             c_int(h), c_int(_is_bf16(x)), _stream()), "moe_gather")
    return QuantActs(xq, sf, (ws.rows_pad, h), x.dtype)


def gemm_grouped(x, weight, ws: MoeWorkspace, experts_local: int, alpha=None, bias=None, w_sf=None):
    """Expert GEMM over the padded rows: ``x`` 16-bit ``[rows_pad, K]`` or ``QuantActs``; ``weight``
    ``[E_local * N, K]`` (16-bit) or packed NVFP4 ``[E_local * N, K/2]`` with atom scales ``w_sf``."""
    wsx = Workspace.get(weight.device)
    if isinstance(x, QuantActs):
        n = weight.shape[0] // experts_local
        k = weight.shape[1] * 2
        out = torch.empty(ws.rows_pad, n, dtype=x.dtype, device=weight.device)
        _check(lib().telb_gemm_nvfp4_grouped(_p(x.xq), _p(x.sf), _p(weight), _p(w_sf), _p(out), c_int(ws.rows_pad), c_int(n), c_int(k),
                                             c_int(experts_local), _p(ws.tile_expert), _p(alpha),
                                             c_int(1 if x.dtype == torch.bfloat16 else 0), _p(wsx.status), _stream()),
               "gemm_nvfp4_grouped")
        return out
    n = weight.shape[0] // experts_local
    k = weight.shape[1]
    out = torch.empty(ws.rows_pad, n, dtype=x.dtype, device=x.device)
    if x.dtype == torch.float32:
        _check(lib().telb_gemm_f32_grouped(_p(x), _p(weight), _p(out), c_int(ws.rows_pad), c_int(n), c_int(k), _p(ws.tile_expert), _p(bias),
                                           _stream()), "gemm_f32_grouped")
        return out
    _check(lib().telb_gemm_f16_grouped(_p(x), _p(weight), _p(out), c_int(ws.rows_pad), c_int(n), c_int(k), c_int(experts_local),
                                       _p(ws.tile_expert), _p(alpha), _p(bias), c_int(_is_bf16(x)), _p(wsx.status), _stream()),
           "gemm_f16_grouped")
    return out


def gemm_grouped_swiglu(x: "QuantActs", weight, ws: MoeWorkspace, experts_local: int, alpha, w_sf, out_scale: torch.Tensor) -> "QuantActs":
    """Expert gate/up GEMM over the padded rows whose epilogue applies SwiGLU and quantises to NVFP4 for the second expert GEMM
    (each expert's ``2 * inter`` weight rows alternate gate / up in blocks of 64).  Padding rows are left unwritten."""
    n = weight.shape[0] // experts_local
    k = weight.shape[1] * 2
    inter = n // 2
    L = lib()
    L.telb_nvfp4_sf_bytes.restype = c_ll
    xq = torch.empty(ws.rows_pad, inter // 2, dtype=torch.uint8, device=weight.device)
    sf = _sf_buffer(L.telb_nvfp4_sf_bytes(c_ll(ws.rows_pad), c_int(inter)), inter, weight.device)
    wsx = Workspace.get(weight.device)
    _check(L.telb_gemm_nvfp4_grouped_swiglu(_p(x.xq), _p(x.sf), _p(weight), _p(w_sf), _p(xq), _p(sf), _p(out_scale), c_int(ws.rows_pad),
                                            c_int(n), c_int(k), c_int(experts_local), _p(ws.tile_expert), _p(alpha),
                                            c_int(1 if x.dtype == torch.bfloat16 else 0), _p(wsx.status), _stream()),
           "gemm_nvfp4_grouped_swiglu")
    return QuantActs(xq, sf, (ws.rows_pad, inter), x.dtype)


def moe_combine(y: torch.Tensor, ws, topk_w: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out[t] = Σ_k w[t,k] · y[ws.dst_row[t*K + k]]`` (slots with a negative row contribute nothing)."""
    t, k = topk_w.shape
    if out is None:
        out = torch.empty(t, y.shape[1], dtype=y.dtype, device=y.device)
    _check(lib().telb_moe_combine(_p(y), _p(ws.dst_row), _p(topk_w), _p(out), c_int(t), c_int(k), c_int(y.shape[1]),
                                  c_int(_is_bf16(y)), _stream()), "moe_combine")
    return out


# ---- recurrent layers ---------------------------------------------------------------------------


def causal_conv1d(x, weight, bias, conv_state, meta: StepMeta, activation=True):
    x = x.contiguous()
    t, c = x.shape
    w = weight.reshape(c, -1).contiguous()
    out = torch.empty_like(x)
    assert conv_state.is_contiguous() and conv_state.dtype == x.dtype
    _check(lib().telb_causal_conv1d(_p(x), _p(w), _p(bias), _p(conv_state), _p(out), _p(meta.seq_ids), _p(meta.q_start),
                                    _p(meta.q_len), _p(meta.past_len), _p(meta.slot_ids), c_int(t), c_int(meta.num_seqs), c_int(c),
                                    c_int(w.shape[1]), c_int(int(activation)), c_int(_is_bf16(x)), _stream()), "causal_conv1d", 2)
    return out


_SSM_SCRATCH = {}


SSD_TC_MIN_Q = 64        # steps whose longest sequence has at least this many new rows take the tensor-core chunk scan


def ssm_scan(x, dt, A, B, C, D, dt_bias, ssm_state, meta: StepMeta, z=None, dt_softplus=True, dt_limit=0.0):
    x, dt, B, C = x.contiguous(), dt.contiguous(), B.contiguous(), C.contiguous()
    t, nh, hd = x.shape
    y = torch.empty_like(x)
    assert ssm_state.dtype == torch.float32 and ssm_state.is_contiguous()
    if (meta.max_q_len >= SSD_TC_MIN_Q and hd == 64 and B.shape[-1] == 128 and os.environ.get("TELB_DISABLE_SSD_TC", "0") != "1"):
        # prefill: chunked state-space-duality scan on the tensor cores (csrc/kernels/ssd_tc5.cu)
        ws = Workspace.get(x.device)
        _check(lib().telb_ssd_chunk_scan(_p(x), _p(dt), _p(A.float().contiguous()), _p(B), _p(C), _p(D.float().contiguous()),
                                         _p(dt_bias.float().contiguous()), _p(z.contiguous() if z is not None else None), _p(ssm_state), _p(y),
                                         _p(meta.q_start), _p(meta.q_len), _p(meta.past_len), _p(meta.slot_ids), c_int(meta.num_seqs), c_int(t),
                                         c_int(nh), c_int(hd), c_int(B.shape[-1]), c_int(B.shape[1]), c_int(int(dt_softplus)),
                                         c_float(dt_limit), c_int(_is_bf16(x)), _p(ws.status), _stream()), "ssd_chunk_scan")
        return y
    scratch = None
    if meta.max_q_len >= 256:       # long prefill chunk: parallel segments need per-segment states (see recurrent.cu)
        segs = (meta.max_q_len + 127) // 128
        need = meta.num_seqs * nh * segs * (hd * B.shape[-1] + 1)
        scratch = _SSM_SCRATCH.get(x.device)
        if scratch is None or scratch.numel() < need:
            scratch = _SSM_SCRATCH[x.device] = torch.empty(need, dtype=torch.float32, device=x.device)
    _check(lib().telb_ssm_scan(_p(x), _p(dt), _p(A.float().contiguous()), _p(B), _p(C), _p(D.float().contiguous()),
                               _p(dt_bias.float().contiguous()), _p(z.contiguous() if z is not None else None), _p(ssm_state), _p(y),
                               _p(meta.q_start), _p(meta.q_len), _p(meta.past_len), _p(meta.slot_ids), c_int(meta.num_seqs),
                               c_int(nh), c_int(hd), c_int(B.shape[-1]), c_int(B.shape[1]), c_int(int(dt_softplus)),
                               c_float(dt_limit), c_int(_is_bf16(x)), c_int(meta.max_q_len), _p(scratch),
                               c_ll(scratch.numel() if scratch is not None else 0), _stream()), "ssm_scan", 3 if scratch is not None else 1)
    return y


GDN_TC_MIN_Q = 32        # steps whose longest sequence has at least this many new rows take the tensor-core chunked kernel


def gated_delta_rule(q, k, v, a, b, A_log, dt_bias, state, meta: StepMeta):
    q, k, v, a, b = (t.contiguous() for t in (q, k, v, a, b))
    out = torch.empty_like(v)
    assert state.dtype == torch.float32 and state.is_contiguous()
    if (meta.max_q_len >= GDN_TC_MIN_Q and q.shape[2] == 128 and v.shape[2] == 128 and os.environ.get("TELB_DISABLE_GDN_TC", "0") != "1"):
        # prefill: chunked (64-token) delta rule with the matrix products on the tensor cores (csrc/kernels/gdn_tc5.cu)
        ws = Workspace.get(q.device)
        _check(lib().telb_gdn_chunk_prefill(_p(q), _p(k), _p(v), _p(a), _p(b), _p(A_log.float().contiguous()), _p(dt_bias.float().contiguous()),
                                            _p(state), _p(out), _p(meta.q_start), _p(meta.q_len), _p(meta.past_len), _p(meta.slot_ids),
                                            c_int(meta.num_seqs), c_int(q.shape[0]), c_int(q.shape[1]), c_int(v.shape[1]), c_int(q.shape[2]),
                                            c_int(v.shape[2]), c_int(_is_bf16(q)), _p(ws.status), _stream()), "gdn_chunk_prefill")
        return out
    _check(lib().telb_gated_delta_rule(_p(q), _p(k), _p(v), _p(a), _p(b), _p(A_log.float().contiguous()),
                                       _p(dt_bias.float().contiguous()), _p(state), _p(out), _p(meta.q_start), _p(meta.q_len),
                                       _p(meta.past_len), _p(meta.slot_ids), c_int(meta.num_seqs), c_int(q.shape[1]), c_int(v.shape[1]),
                                       c_int(q.shape[2]), c_int(v.shape[2]), c_int(_is_bf16(q)), _stream()), "gated_delta_rule")
    return out


class MlstmParams(ctypes.Structure):
    """Host mirror of ``MlstmParams`` (``csrc/kernels/mlstm_common.cuh``)."""
    _fields_ = [(n, c_vp) for n in ("qkvg", "gates", "state", "norm_state", "norm_w", "out", "o32", "n_next", "q_start", "q_len", "past_len",
                                    "slot_ids", "status")] + \
               [(n, c_int) for n in ("ld", "ldg", "heads", "dk", "dv", "k_off", "v_off", "g_off", "dv_real")] + \
               [(n, c_float) for n in ("scale", "cap", "eps")]


MLSTM_TC_MIN_Q = 16      # steps whose longest sequence has at least this many new rows take the chunked tensor-core kernel


def mlstm(qkvg, gates, norm_w, state, norm_state, meta: StepMeta, scale: float, cap: float, eps: float, dv_real: int,
          kernel: Optional[str] = None) -> torch.Tensor:
    """See :func:`ops.mlstm`.  Steps of one row per sequence run the fused decode kernel, longer ones the chunked tensor-core kernel
    (16-bit rows) or the row-by-row walk; ``kernel`` forces ``"decode"``, ``"chunk"`` or ``"scan"``."""
    qkvg = qkvg.contiguous()
    t = qkvg.shape[0]
    _, n, dk, dv = state.shape
    assert state.dtype == norm_state.dtype == norm_w.dtype == gates.dtype == torch.float32
    assert state.is_contiguous() and norm_state.is_contiguous() and gates.stride(1) == 1
    assert qkvg.shape[1] == 2 * n * (dk + dv) and norm_state.shape[1:] == (n, dk + 1) and norm_w.numel() == n * dv and gates.shape[1] >= 2 * n
    chunk_ok = qkvg.dtype != torch.float32 and dk in (64, 128) and dv % 128 == 0
    if kernel is None:
        if meta.max_q_len == 1 and dv <= 1024:
            kernel = "decode"
        else:
            kernel = "chunk" if chunk_ok and meta.max_q_len >= MLSTM_TC_MIN_Q else "scan"
    if (kernel == "decode" and meta.max_q_len != 1) or (kernel == "chunk" and not chunk_ok):
        raise ValueError(f"the {kernel} kernel does not cover this step")
    out = torch.empty(t, n * dv, dtype=qkvg.dtype, device=qkvg.device)
    o32 = nn = None
    if kernel == "scan" or (kernel == "chunk" and dv != 128):
        o32 = torch.empty(t, n, dv, dtype=torch.float32, device=qkvg.device)
        nn = torch.empty(meta.num_seqs, n, dk + 1, dtype=torch.float32, device=qkvg.device)
    ptr = lambda x: None if x is None else _p(x).value
    p = MlstmParams(*[ptr(x) for x in (qkvg, gates, state, norm_state, norm_w, out, o32, nn, meta.q_start, meta.q_len, meta.past_len,
                                       meta.slot_ids, Workspace.get(qkvg.device).status)],
                    qkvg.shape[1], gates.stride(0), n, dk, dv, n * dk, 2 * n * dk, n * (2 * dk + dv), dv_real, scale, cap, eps)
    code = _dtype_code(qkvg)
    L, ref_p = lib(), ctypes.byref(p)
    if kernel == "decode":
        _check(L.telb_mlstm_decode(ref_p, c_int(meta.num_seqs), c_int(code), _stream()), "mlstm_decode")
    elif kernel == "chunk":
        _check(L.telb_mlstm_chunk(ref_p, c_int(meta.num_seqs), c_int(t), c_int(code), _stream()), "mlstm_chunk", 1 if dv == 128 else 2)
    else:
        _check(L.telb_mlstm_scan(ref_p, c_int(meta.num_seqs), c_int(t), c_int(code), _stream()), "mlstm_scan", 2)
    return out


class LightningParams(ctypes.Structure):
    """Host mirror of ``LightningParams`` (``csrc/kernels/lightning_common.cuh``)."""
    _fields_ = [(n, c_vp) for n in ("rows", "act", "powers", "state", "norm_w", "out", "sums", "carry", "q_start", "q_len", "past_len", "slot_ids", "status")] + \
               [(n, c_int) for n in ("ld", "heads", "dk", "dv", "k_off", "v_off", "g_off", "n_powers", "tokens", "num_seqs", "segments", "seg_chunks")]


LIGHTNING_TC_MIN_Q = 16      # steps whose longest sequence has at least this many new rows take the chunked tensor-core kernel


def _lightning_segments(meta: StepMeta, tiles: int) -> Tuple[int, int]:
    """``(segments, chunks per segment)`` of the longest sequence: few (sequence, head, value tile) triples are cut until about every SM has one."""
    chunks = (meta.max_q_len + 127) // 128
    want = max(1, 148 // tiles)
    if want < 2 or chunks < 4:
        return 1, chunks
    per = max(2, (chunks + want - 1) // want)
    return (chunks + per - 1) // per, per


def lightning(rows, norm_w, powers, state, meta: StepMeta, kernel: Optional[str] = None, segments: Optional[Tuple[int, int]] = None):
    """See :func:`ops.lightning`.  Steps of one row per sequence run the decode kernel, longer ones the chunked tensor-core kernel (bf16) or
    the walk row by row; ``kernel`` forces ``"step"``, ``"chunk"`` or ``"walk"``."""
    rows = rows.contiguous()
    t = rows.shape[0]
    _, n, dk, dv = state.shape
    f32, dev = torch.float32, rows.device
    if rows.dtype not in (torch.bfloat16, f32):
        raise TypeError(f"lightning: un-normed rows leave in bf16 or fp32, not {rows.dtype}")
    assert state.dtype == norm_w.dtype == powers.dtype == f32 and state.is_contiguous() and powers.is_contiguous()
    assert rows.shape[1] == 2 * n * (dk + dv) and norm_w.numel() == n * dv and powers.shape[0] == n
    chunk_ok = rows.dtype == torch.bfloat16 and dk in (64, 128) and powers.shape[1] > 128
    if kernel is None:
        kernel = "step" if meta.max_q_len == 1 else "chunk" if chunk_ok and meta.max_q_len >= LIGHTNING_TC_MIN_Q else "walk"
    if (kernel == "step" and meta.max_q_len != 1) or (kernel == "chunk" and not chunk_ok):
        raise ValueError(f"the {kernel} kernel does not cover this step")
    out = torch.empty(t, n * dv, dtype=rows.dtype, device=dev)
    sums = torch.empty(t, n * dv // 32, dtype=f32, device=dev)
    act = carry = None
    segs, per, launches = 1, 0, 1
    if kernel == "chunk":
        segs, per = segments or _lightning_segments(meta, meta.num_seqs * n * (dv // 128))
        act = torch.empty(t, n * (2 * dk + dv), dtype=rows.dtype, device=dev)
        if segs > 1:
            carry = torch.empty(meta.num_seqs, n, segs, dk, dv, dtype=f32, device=dev)
        launches = 2 if segs == 1 else 4
    ptr = lambda x: None if x is None else _p(x).value
    p = LightningParams(*[ptr(x) for x in (rows, act, powers, state, norm_w, out, sums, carry, meta.q_start, meta.q_len, meta.past_len, meta.slot_ids,
                                           Workspace.get(dev).status)],
                        rows.shape[1], n, dk, dv, n * dk, 2 * n * dk, n * (2 * dk + dv), powers.shape[1], t, meta.num_seqs, segs, per)
    L, ref_p = lib(), ctypes.byref(p)
    if kernel == "chunk":
        _check(L.telb_lightning_chunk(ref_p, _stream()), "lightning_chunk", launches)
    else:
        f = L.telb_lightning_step if kernel == "step" else L.telb_lightning_walk
        _check(f(ref_p, c_int(_dtype_code(rows)), _stream()), f"lightning_{kernel}")
    return out, sums


class ChannelDeltaParams(ctypes.Structure):
    """Host mirror of ``ChannelDeltaParams`` (``csrc/kernels/channel_delta.cu``)."""
    _fields_ = [(n, c_vp) for n in ("qkv", "decay", "gate", "beta", "conv_w", "a_log", "decay_bias", "norm_w", "conv_state", "state", "blocks",
                                    "v_blocks", "o", "out", "q_start", "q_len", "past_len", "slot_ids", "seq_ids", "status")] + \
               [(n, c_int) for n in ("tokens", "num_seqs", "heads", "kv_heads", "dk", "dv", "dk_real", "dv_real", "taps", "channels", "ld_decay", "ld_gate",
                                     "gate_f32", "ld_qkv", "ld_beta", "ld_out", "head_decay", "gate_silu")] + [("eps", c_float), ("mult", c_float)]


def _pitched(x: torch.Tensor) -> torch.Tensor:
    """``x`` itself when its rows are contiguous and 16-byte aligned (they may lie further apart), else a copy."""
    return x if x.stride(1) == 1 and x.stride(0) % 8 == 0 and x.storage_offset() % 8 == 0 else x.contiguous()


def channel_delta(qkv, decay, gate, beta, conv_w, a_log, decay_bias, norm_w, conv_state, state, meta: StepMeta, spec, eps: float,
                  kernel: Optional[str] = None, out: Optional[torch.Tensor] = None, mult: float = 1.0) -> torch.Tensor:
    """See :func:`ops.channel_delta`.  Steps of one row per sequence run the fused decode kernel, longer ones the walk over rows;
    ``kernel`` forces ``"decode"`` or ``"walk"``."""
    qkv = _pitched(qkv)
    t, ch = qkv.shape
    n, nk, dk, dv = spec.num_heads, spec.num_kv_heads, spec.k_pad, spec.v_pad
    f32 = torch.float32
    assert ch == spec.conv_dim and conv_w.shape == (ch, spec.conv_kernel) and conv_w.dtype == conv_state.dtype == qkv.dtype
    assert state.dtype == decay.dtype == beta.dtype == a_log.dtype == decay_bias.dtype == norm_w.dtype == f32
    assert state.shape[1:] == (n, dk, dv) and state.is_contiguous() and conv_state.is_contiguous() and conv_w.is_contiguous()
    assert decay.shape == (t, n if spec.head_decay else n * dk) and decay_bias.numel() == decay.shape[1]
    assert gate.shape == (t, n * dv) and beta.shape == (t, n) and decay.stride(1) == gate.stride(1) == beta.stride(1) == 1
    if gate.dtype not in (qkv.dtype, f32) or (not spec.head_decay and decay.stride(0) % 4) or gate.stride(0) % 4:
        raise TypeError(f"channel_delta: gate {gate.dtype} for {qkv.dtype} rows, row pitches {decay.stride(0)}, {gate.stride(0)}")
    decode_ok = meta.max_q_len == 1 and dk <= 128 and dv <= 128
    if kernel is None:
        kernel = "decode" if decode_ok else "walk"
    if kernel == "decode" and not decode_ok:
        raise ValueError("the decode kernel does not cover this step")
    dev = qkv.device
    if out is None:
        out = torch.empty(t, n * dv, dtype=qkv.dtype, device=dev)
    assert out.shape == (t, n * dv) and out.dtype == qkv.dtype and out.stride(1) == 1 and out.stride(0) % 8 == 0
    blocks = v_blocks = o = None
    if kernel == "walk":                       # blocks of four tokens, counted from the start of every portion
        nb = t // 4 + meta.num_seqs + 1
        blocks, v_blocks = torch.empty(nb, n, (8 if spec.head_decay else 13) * dk + 32, dtype=f32, device=dev), torch.empty(nb, n, dv, 4, dtype=qkv.dtype, device=dev)
        o = torch.empty(t, n * dv, dtype=qkv.dtype, device=dev)
    ptr = lambda x: None if x is None else _p(x).value
    p = ChannelDeltaParams(*[ptr(x) for x in (qkv, decay, gate, beta, conv_w, a_log, decay_bias, norm_w, conv_state, state, blocks, v_blocks, o, out,
                                              meta.q_start, meta.q_len, meta.past_len, meta.slot_ids, meta.seq_ids, Workspace.get(dev).status)],
                           t, meta.num_seqs, n, nk, dk, dv, spec.head_k_dim, spec.head_v_dim, spec.conv_kernel, ch, decay.stride(0), gate.stride(0),
                           int(gate.dtype == f32), qkv.stride(0), beta.stride(0), out.stride(0), int(spec.head_decay), int(spec.silu_gate), eps, mult)
    launches = (1 if kernel == "decode" else 4) + int(spec.conv_kernel > 1 and (kernel == "walk" or n != nk))
    _check(lib().telb_channel_delta(ctypes.byref(p), c_int(int(kernel == "decode")), c_int(_dtype_code(qkv)), _stream()), "channel_delta", launches)
    return out


# ---- attention with cache rows of its own ---------------------------------------------------------


def unit_kv_write(qkv, kv_layer, meta: StepMeta, temperature, num_q_heads: int, num_kv_heads: int, head_dim: int, real_dim: int, eps: float):
    qkv = qkv.contiguous()
    t = qkv.shape[0]
    assert kv_layer.is_contiguous() and kv_layer.dtype == qkv.dtype and kv_layer.shape[1:3] == (2, num_kv_heads) and kv_layer.shape[4] == head_dim
    q = torch.empty(t, num_q_heads, head_dim, dtype=qkv.dtype, device=qkv.device)
    _check(lib().telb_unit_kv_write(
        _p(qkv), _p(q), _p(kv_layer), _p(temperature), _p(meta.positions), _p(meta.seq_ids), _p(meta.q_start), _p(meta.past_len), _p(meta.page_table),
        c_int(t), c_int(meta.page_table.shape[1]), c_int(meta.page_size), c_int(num_q_heads), c_int(num_kv_heads), c_int(head_dim), c_int(real_dim),
        c_float(eps), c_int(_dtype_code(qkv)), _stream()), "unit_kv_write")
    return q


class TurnedKvParams(ctypes.Structure):
    """Host mirror of ``TurnedKvParams`` (``csrc/kernels/latent.cu``)."""
    _fields_ = [(n, c_vp) for n in ("rows", "q_out", "kv", "key_table", "value_table", "q_norm", "k_norm", "positions", "seq_ids", "q_start", "past_len",
                                    "page_table")] + \
               [(n, c_int) for n in ("ld", "tokens", "max_pages", "page_size", "hq", "hkv", "d", "real")] + [("eps", c_float)]


def turned_kv_write(rows, kv_layer, meta: StepMeta, key_table, value_table, q_norm, k_norm, spec, eps: float):
    rows = _pitched(rows)
    t, hq, hkv, d = rows.shape[0], spec.num_heads, spec.num_kv_heads, spec.pad
    f32 = torch.float32
    assert rows.shape[1] == (hq + 2 * hkv) * d and kv_layer.is_contiguous() and kv_layer.dtype == rows.dtype
    assert kv_layer.shape[1:] == (2, hkv, meta.page_size, d)
    assert all(x.dtype == f32 and x.is_contiguous() for x in (key_table, value_table, q_norm, k_norm))
    assert key_table.shape[1] == value_table.shape[1] == d and q_norm.numel() == hq * d and k_norm.numel() == hkv * d
    q = torch.empty(t, hq, d, dtype=rows.dtype, device=rows.device)
    p = TurnedKvParams(*[_p(x).value for x in (rows, q, kv_layer, key_table, value_table, q_norm, k_norm, meta.positions, meta.seq_ids, meta.q_start,
                                               meta.past_len, meta.page_table)],
                       rows.stride(0), t, meta.page_table.shape[1], meta.page_size, hq, hkv, d, spec.head_dim, eps)
    _check(lib().telb_turned_kv_write(ctypes.byref(p), c_int(_dtype_code(rows)), _stream()), "turned_kv_write")
    return q


MIXED_DECODE_COLUMNS = 64       # sequences with at most this many (row, head) pairs in a step run the token-major kernel


class RowSplit:
    """A step's sequences by how many rows they bring: ``short`` (up to ``limit``) and ``long``, each ``(q_start, q_len, past_len, page_table,
    sequences, most rows, longest sequence)`` over the rows of the whole step, or None.  Built once per step."""

    def __init__(self, meta: StepMeta, limit: int, device):
        self.key = ("rows", limit)
        everything = (meta.q_start, meta.q_len, meta.past_len, meta.page_table, meta.num_seqs, meta.max_q_len, meta.max_seq_len)
        self.short = self.long = None
        if meta.max_q_len <= limit:
            self.short = everything
            return
        lens, start = meta.lengths(), [0]
        for q, _ in lens:
            start.append(start[-1] + q)
        parts = [[i for i, (q, _) in enumerate(lens) if 0 < q <= limit], [i for i, (q, _) in enumerate(lens) if q > limit]]
        if len(parts[1]) == len(lens):
            self.long = everything
            return
        out = []
        for part in parts:
            if not part:
                out.append(None)
                continue
            arr = torch.tensor([[start[i] for i in part], [lens[i][0] for i in part], [lens[i][1] for i in part]], dtype=torch.int32, device=device)
            table = meta.page_table.index_select(0, torch.tensor(part, dtype=torch.int64, device=device))
            out.append((arr[0], arr[1], arr[2], table, len(part), max(lens[i][0] for i in part), max(sum(lens[i]) for i in part)))
        self.short, self.long = out


def _row_split(meta: StepMeta, limit: int, device) -> RowSplit:
    for p in meta.plans or ():
        if p.key == ("rows", limit):
            return p
    p = RowSplit(meta, limit, device)
    meta.plans = (meta.plans or ()) + (p,)
    return p


class MixedKvParams(ctypes.Structure):
    """Host mirror of ``MixedKvParams`` (``csrc/kernels/mixed_heads.cu``)."""
    _fields_ = [(n, c_vp) for n in ("rows", "first", "q_out", "kv", "mix", "share", "seq_ids", "q_start", "past_len", "page_table")] + \
               [(n, c_ll) for n in ("ld", "ld_first")] + [(n, c_int) for n in ("tokens", "max_pages", "page_size", "hq", "hkv", "d", "halves", "d_first")]


def _mixed_tc(spec, dtype, page_size: int) -> bool:
    """Whether the tensor-core kernels take this layer."""
    return dtype == torch.bfloat16 and page_size == 64 and spec.pad in (64, 128) and spec.num_kv_heads * spec.pad <= 512


def _mixed_plan(meta: StepMeta, heads: int, device) -> RowSplit:
    return _row_split(meta, max(1, MIXED_DECODE_COLUMNS // heads), device)


def mixed_kv_write(rows, kv_layer, meta: StepMeta, mix, first, share, spec):
    """See :func:`ops.mixed_kv_write`; 16-bit wide queries come as high | low halves where the kernels behind can use both."""
    t, n, g, d = rows.shape[0], spec.num_heads, spec.num_kv_heads, spec.pad
    rows = _pitched(rows)
    assert rows.shape[1] >= (n + 2 * g) * d and kv_layer.is_contiguous() and kv_layer.dtype == rows.dtype and kv_layer.shape[1:] == (2, g, meta.page_size, d)
    assert mix.dtype == torch.float32 and mix.is_contiguous() and mix.shape == (n, n) and share.dtype == torch.float32
    if first is not None:
        first = _pitched(first)
        assert first.dtype == rows.dtype and first.shape[0] == t and first.shape[1] % (8 * g) == 0
    halves = 1
    if _mixed_tc(spec, rows.dtype, meta.page_size) and (g * d <= 256 or _mixed_plan(meta, n, rows.device).long is None):
        halves = 2
    q = torch.empty(t, n, halves * g * d, dtype=rows.dtype, device=rows.device)
    p = MixedKvParams(*[None if x is None else _p(x).value for x in (rows, first, q, kv_layer, mix, share, meta.seq_ids, meta.q_start, meta.past_len, meta.page_table)],
                      rows.stride(0), 0 if first is None else first.stride(0), t, meta.page_table.shape[1], meta.page_size, n, g, d, halves, 0 if first is None else first.shape[1] // g)
    _check(lib().telb_mixed_kv_write(ctypes.byref(p), c_int(_dtype_code(rows)), _stream()), "mixed_kv_write")
    return q


def mixed_attention(q, kv_layer, meta: StepMeta, slopes, gate, spec, kernel: Optional[str] = None, splits: Optional[int] = None, tile: Optional[int] = None):
    """See :func:`ops.mixed_attention`.  Sequences with few rows run the token-major kernel, prompt portions the row-major one (``kernel``
    forces ``"decode"``, ``"prefill"`` or ``"simt"`` for all); fp32 rows and sizes without a tensor-core form run on the CUDA cores."""
    if meta.tree_mask is not None:
        raise ValueError("mixed attention covers causal windows only")
    (t, n, width), g, d, dev = q.shape, spec.num_kv_heads, spec.pad, q.device
    halves = width // (g * d)
    out = torch.empty(t, n * d, dtype=q.dtype, device=dev)
    ld_gate = 0
    if gate is not None:
        assert gate.shape == (t, n * d) and gate.dtype == q.dtype and gate.stride(1) == 1
        ld_gate = gate.stride(0)
    assert slopes.dtype == torch.float32 and slopes.numel() == n and spec.window >= 1
    if kernel == "simt" or not _mixed_tc(spec, q.dtype, meta.page_size):
        q = q[:, :, :g * d].contiguous()
        _check(lib().telb_mixed_attention_simt(
            _p(q), _p(kv_layer), _p(out), _p(meta.q_start), _p(meta.past_len), _p(meta.seq_ids), _p(meta.page_table), c_int(t), c_int(meta.page_table.shape[1]),
            c_int(meta.page_size), c_int(n), c_int(g), c_int(d), c_float(spec.scale), c_int(spec.window), _p(slopes), _p(gate), c_ll(ld_gate),
            c_int(_dtype_code(q)), _stream()), "mixed_attention_simt")
        return out
    everything = (meta.q_start, meta.q_len, meta.past_len, meta.page_table, meta.num_seqs, meta.max_q_len, meta.max_seq_len)
    if kernel is None:
        plan = _mixed_plan(meta, n, dev)
        short, long = plan.short, plan.long
    else:
        short, long = (everything, None) if kernel == "decode" else (None, everything)
    ws = Workspace.get(dev)
    common = lambda s: (_p(q), _p(kv_layer), _p(out), _p(s[0]), _p(s[1]), _p(s[2]), _p(s[3]), c_int(s[4]), c_int(t), c_int(s[5]), c_int(kv_layer.shape[0]),
                        c_int(s[3].shape[1]), c_int(n), c_int(g), c_int(d), c_int(halves), c_float(spec.scale), c_int(spec.window), _p(slopes), _p(gate), c_ll(ld_gate))
    if long is not None:
        _check(lib().telb_mixed_attention_prefill(*common(long), _p(ws.status), _stream()), "mixed_attention_prefill")
    if short is not None:
        nc = 16 if short[5] * n <= 16 else 32
        sp, tl = _latent_splits(short[4] * ((short[5] * n + nc - 1) // nc), min(short[6], spec.window + short[5] + 63), nc)
        sp, tl = splits or sp, tile or tl
        _check(lib().telb_mixed_attention_decode(*common(short), c_int(sp), c_int(tl), _p(ws.attn_ws), c_ll(ws.attn_ws.numel()), _p(ws.status), _stream()),
               "mixed_attention_decode", 2 if sp > 1 else 1)
    return out


def latent_write(rows, kv_layer, meta: StepMeta, cos_sin, norm_w, spec, eps: float):
    rows = rows.contiguous()
    n = spec.num_heads
    assert rows.shape[1] == n * (spec.k_pad + spec.rot_pad) + spec.pad and norm_w.dtype == torch.float32 and norm_w.numel() == spec.rank_pad
    assert kv_layer.is_contiguous() and kv_layer.dtype == rows.dtype and tuple(kv_layer.shape[1:]) == (1, 1, meta.page_size, spec.pad)
    _check(lib().telb_latent_write(
        _p(rows), _p(kv_layer), _p(cos_sin), _p(norm_w), _p(meta.positions), _p(meta.seq_ids), _p(meta.q_start), _p(meta.past_len), _p(meta.page_table),
        c_int(rows.shape[0]), c_int(meta.page_table.shape[1]), c_int(meta.page_size), c_int(n), c_int(spec.k_pad), c_int(spec.rot_pad),
        c_int(spec.rank_pad), c_int(spec.rank), c_int(spec.rot_dim), c_int(cos_sin.shape[1]), c_float(eps), c_int(_dtype_code(rows)), _stream()), "latent_write")
    return rows


def head_linear(x, weight, heads: int, x_col: int = 0, tail_col: int = -1, tail: int = 0) -> torch.Tensor:
    """``y[t, h] = weight[h] · x[t, h]`` for ``weight [H, N, K]`` and the ``H · K`` columns of ``x [T, ld]`` from ``x_col`` on; with ``tail``,
    ``x``'s columns from ``tail_col`` on (``tail`` per head) follow each head's result.  ``[T, H, N + tail]``."""
    t, (h, n, k) = x.shape[0], weight.shape
    assert h == heads and x.is_contiguous() and weight.is_contiguous() and x.dtype == weight.dtype
    y = torch.empty(t, h, n + tail, dtype=x.dtype, device=x.device)
    base, es = x.data_ptr(), x.element_size()
    _p(x)
    _check(lib().telb_head_linear(c_vp(base + x_col * es), _p(weight), _p(y), c_vp(base + max(tail_col, 0) * es), c_int(t), c_int(h), c_int(n), c_int(k),
                                  c_int(tail), c_int(x.shape[1]), c_int(x.shape[1]), c_int(h * (n + tail)), c_int(n + tail), c_int(_dtype_code(x)),
                                  _p(Workspace.get(x.device).status), _stream()), "head_linear")
    return y


LATENT_FOLDED_COLUMNS = 128      # sequences with at most this many (row, head) pairs in a step read the cached latents directly


class LatentPlan:
    """How a step's sequences run in latent attention: a few rows per sequence against the cached latents themselves (the key expansion
    folded into the query), prompt portions over keys and values expanded for them.  Built once per step."""

    def __init__(self, meta: StepMeta, heads: int, device, force: Optional[str]):
        self.key = (heads, force)
        limit = {None: max(1, LATENT_FOLDED_COLUMNS // heads), "folded": 1 << 30, "expanded": 0}[force]
        self.rows = self.expand = None                    # rows of the folded sequences (None: all rows), arrays of the expanded ones
        self.folded = (meta.q_start, meta.q_len, meta.past_len, meta.page_table, meta.seq_ids, meta.num_tokens, meta.num_seqs, meta.max_q_len)
        self.max_seq_len = meta.max_seq_len
        if meta.max_q_len <= limit:
            return
        lens = meta.lengths()
        i32 = dict(dtype=torch.int32, device=device)
        start = [0]
        for q, _ in lens:
            start.append(start[-1] + q)
        short = [i for i, (q, _) in enumerate(lens) if 0 < q <= limit]
        long = [i for i, (q, _) in enumerate(lens) if q > limit]
        kv_start, kv_rows = [], 0
        for i in long:
            kv_start.append(kv_rows)
            kv_rows += sum(lens[i])
        packed = torch.tensor([[start[i] for i in long], [lens[i][0] for i in long], [lens[i][1] for i in long], kv_start], **i32)
        table = meta.page_table if len(long) == len(lens) else meta.page_table.index_select(0, torch.tensor(long, dtype=torch.int64, device=device))
        self.expand = (packed[0], packed[1], packed[2], packed[3], table.contiguous(), len(long), max(lens[i][0] for i in long), kv_rows,
                       max(sum(lens[i]) for i in long))
        if not short:
            self.folded = None
            return
        rows, q_start, seq_ids = [], [], []
        for n, i in enumerate(short):
            q_start.append(len(rows))
            rows += range(start[i], start[i] + lens[i][0])
            seq_ids += [n] * lens[i][0]
        self.rows = torch.tensor(rows, dtype=torch.int64, device=device)
        arr = torch.tensor([q_start, [lens[i][0] for i in short], [lens[i][1] for i in short]], **i32)
        table = meta.page_table.index_select(0, torch.tensor(short, dtype=torch.int64, device=device))
        self.folded = (arr[0], arr[1], arr[2], table, torch.tensor(seq_ids, **i32), len(rows), len(short), max(lens[i][0] for i in short))
        self.max_seq_len = max(sum(lens[i]) for i in short)


def _latent_plan(meta: StepMeta, heads: int, device, force: Optional[str]) -> LatentPlan:
    for p in meta.plans or ():
        if p.key == (heads, force):
            return p
    p = LatentPlan(meta, heads, device, force)
    meta.plans = (meta.plans or ()) + (p,)
    return p


def _latent_splits(blocks: int, max_seq_len: int, columns: int) -> Tuple[int, int]:
    """``(splits, rows per tile)`` of the cached rows for ``blocks`` (column block, sequence) pairs, so that the CTAs come out near whole
    waves.  Costs in the time of a one-page tile; a two-page tile takes little longer than that while an SM has a CTA to itself."""
    best, cost = (1, 128), None
    for tile, slots, unit in ((64, 296 if columns == 16 else 148, 1.7 if columns == 16 else 1.0), (128, 148, 1.0)):
        tiles = max(1, (max_seq_len + tile - 1) // tile)
        for s in range(1, min(tiles, 64) + 1):
            ctas = blocks * s
            waves = (ctas + slots - 1) // slots
            alone = ctas <= 148                              # one CTA per SM: it does not share the tensor cores
            c = waves * ((tiles + s - 1) // s * ((0.9 if tile == 64 else 1.0) if alone else unit) + 1.0) + (1.0 + s / 32 if s > 1 else 0.0)
            if cost is None or c < cost - 1e-9:
                best, cost = (s, tile), c
    return best


def latent_attention(rows, kv_layer, meta: StepMeta, kv_up, key_up_t, spec, kernel: Optional[str] = None) -> torch.Tensor:
    """See :func:`ops.latent_attention`.  16-bit steps run the tcgen05 kernels where the sizes fit (``kernel`` forces ``"folded"`` or
    ``"expanded"``, ``"folded-64"`` / ``"folded-128"`` also the tile); fp32 rows and other sizes run on the CUDA cores (``"simt"``)."""
    force_tile = 0
    if kernel in ("folded-64", "folded-128"):
        kernel, force_tile = "folded", int(kernel[7:])
    if meta.tree_mask is not None:
        raise ValueError("latent attention covers causal masks only")
    t, n, dev = rows.shape[0], spec.num_heads, rows.device
    tc = rows.dtype != torch.float32 and meta.page_size == 64 and spec.rank_pad <= 512 and spec.rot_pad == 64
    expand_ok = tc and spec.v_pad <= 128 and spec.k_pad <= 256 and spec.scale > 0
    if kernel == "simt" or not tc:
        tc, kernel = False, "folded"
    elif not expand_ok:
        if kernel == "expanded":
            raise ValueError("the expanded kernel does not cover this layer")
        kernel = "folded"
    plan = _latent_plan(meta, n, dev, kernel)
    ws = Workspace.get(dev)
    out = None
    if plan.folded is not None:
        q_start, q_len, past_len, table, seq_ids, tf, seqs, max_q = plan.folded
        sub = rows if plan.rows is None else rows[:, :n * (spec.k_pad + spec.rot_pad)].index_select(0, plan.rows)
        q = head_linear(sub, key_up_t, n, 0, n * spec.k_pad, spec.rot_pad)
        o = torch.empty(tf, n, spec.rank_pad, dtype=rows.dtype, device=dev)
        if tc:
            nc = 16 if max_q * n <= 16 else 32
            splits, tile = _latent_splits(seqs * ((max_q * n + nc - 1) // nc), plan.max_seq_len, nc)
            tile = force_tile or tile
            _check(lib().telb_latent_attention_decode(
                _p(q), _p(kv_layer), _p(o), _p(q_start), _p(q_len), _p(past_len), _p(table), c_int(seqs), c_int(tf), c_int(max_q),
                c_int(kv_layer.shape[0]), c_int(table.shape[1]), c_int(n), c_int(spec.rank_pad), c_int(spec.rot_pad), c_float(spec.scale), c_int(splits), c_int(tile),
                _p(ws.attn_ws), c_ll(ws.attn_ws.numel()), c_int(_is_bf16(rows)), _p(ws.status), _stream()), "latent_attention_decode", 2 if splits > 1 else 1)
        else:
            _check(lib().telb_latent_attention_simt(
                _p(q), _p(kv_layer), _p(o), _p(q_start), _p(past_len), _p(seq_ids), _p(table), c_int(tf), c_int(table.shape[1]), c_int(meta.page_size),
                c_int(n), c_int(spec.pad), c_int(spec.rank_pad), c_float(spec.scale), c_int(_dtype_code(q)), _stream()), "latent_attention_simt")
        value_up = kv_up[n * spec.k_pad:].view(n, spec.v_pad, spec.rank_pad)
        res = head_linear(o.view(tf, -1), value_up, n).view(tf, n * spec.v_pad)
        if plan.rows is None:
            return res
        out = torch.empty(t, n * spec.v_pad, dtype=rows.dtype, device=dev)
        out.index_copy_(0, plan.rows, res)
    if plan.expand is not None:
        q_start, q_len, past_len, kv_start, table, seqs, max_q, kv_rows, max_total = plan.expand
        es = rows.element_size()
        latent = torch.empty(kv_rows, spec.rank_pad, dtype=rows.dtype, device=dev)
        rot = torch.empty(kv_rows, spec.rot_pad, dtype=rows.dtype, device=dev)
        _check(lib().telb_latent_gather(_p(kv_layer), _p(latent), _p(rot), _p(kv_start), _p(q_len), _p(past_len), _p(table), c_int(seqs), c_int(max_total),
                                        c_int(table.shape[1]), c_int(meta.page_size), c_int(spec.rank_pad * es), c_int(spec.rot_pad * es), c_int(0), _stream()),
               "latent_gather")
        kv = gemm(latent, kv_up)
        if out is None:
            out = torch.empty(t, n * spec.v_pad, dtype=rows.dtype, device=dev)
        _check(lib().telb_latent_attention_prefill(
            _p(rows), _p(kv), _p(rot), _p(out), _p(q_start), _p(q_len), _p(past_len), _p(kv_start), c_int(seqs), c_int(t), c_int(max_q), c_int(kv_rows),
            c_int(rows.shape[1]), c_int(n), c_int(spec.k_pad), c_int(spec.rot_pad), c_int(spec.v_pad), c_float(spec.scale), c_int(_is_bf16(rows)),
            _p(ws.status), _stream()), "latent_attention_prefill")
    return out


# ---- speculative decoding -------------------------------------------------------------------------


def spec_accept_greedy(target_tokens, tree_tokens, parents, max_path: int, force_len=0):
    b, n = tree_tokens.shape
    dev = tree_tokens.device
    force = None
    if isinstance(force_len, torch.Tensor):
        force = force_len.to(device=dev, dtype=torch.int32).contiguous()
    elif force_len:
        force = torch.full((b,), int(force_len), dtype=torch.int32, device=dev)
    path = torch.zeros(b, max_path, dtype=torch.int32, device=dev)
    plen = torch.empty(b, dtype=torch.int32, device=dev)
    bonus = torch.empty(b, dtype=torch.int32, device=dev)
    tt, tr, pa = target_tokens.to(torch.int32).contiguous(), tree_tokens.to(torch.int32).contiguous(), parents.to(torch.int32).contiguous()
    _check(lib().telb_spec_accept_greedy(_p(tt), _p(tr), _p(pa), _p(path), _p(plen), _p(bonus), c_int(b), c_int(n),
                                         c_int(max_path), _p(force), _stream()), "spec_accept_greedy")
    return path, plen, bonus


def eagle_tree_meta(parents: torch.Tensor, base_pos: torch.Tensor, depth_base: int, pos_offset: int):
    """Packed ancestor mask ``[B * R, ceil(R / 32)]``, depths ``[B, R]`` and positions ``[B * R]`` of a batch of trees given as
    parent tables ``[B, R]`` (parents precede children, ``-1`` = none): one kernel, nothing read back."""
    b, r = parents.shape
    dev = parents.device
    words = (r + 31) // 32
    par = parents.to(torch.int32).contiguous()
    mask = torch.empty(b * r, words, dtype=torch.int32, device=dev)
    depth = torch.empty(b, r, dtype=torch.int32, device=dev)
    pos = torch.empty(b * r, dtype=torch.int32, device=dev)
    base = base_pos.to(device=dev, dtype=torch.int32).contiguous()
    _check(lib().telb_eagle_tree_meta(_p(par), _p(base), _p(mask), _p(depth), _p(pos),
                                      c_int(b), c_int(r), c_int(words), c_int(depth_base), c_int(pos_offset), _stream()), "eagle_tree_meta")
    return mask, depth, pos


def eagle_select_verify(p_sc, p_tok, p_par, p_dep, root, keep: int):
    """The ``keep`` best candidates of each sequence's pool ``[B, P]`` in pool order behind the root: tokens, parents (indices into
    the tree, root = -1 for slot 0) and depths, each ``[B, keep + 1]`` int32."""
    b, pool = p_sc.shape
    dev = p_sc.device
    i32 = lambda t: t.to(device=dev, dtype=torch.int32).contiguous()
    # converted copies stay referenced until the launch: a temporary freed after its pointer was taken would hand its
    # memory to the next conversion
    sc, ptok, ppar, pdep, rt = p_sc.float().contiguous(), i32(p_tok), i32(p_par), i32(p_dep), i32(root)
    tok = torch.empty(b, keep + 1, dtype=torch.int32, device=dev)
    par = torch.empty_like(tok)
    dep = torch.empty_like(tok)
    _check(lib().telb_eagle_select_verify(_p(sc), _p(ptok), _p(ppar), _p(pdep), _p(rt),
                                          c_int(b), c_int(pool), c_int(keep), _p(tok), _p(par), _p(dep), _stream()), "eagle_select_verify")
    return tok, par, dep


def dflash2_grouped_dynamic_conv(hidden, delta, base, residual, block: int, group_size: int):
    """One side of DFlash 2's dynamic grouped convolution over whole proposal blocks (16-bit in, 16-bit out)."""
    assert hidden.dtype in (torch.float16, torch.bfloat16)
    h, d, b = hidden.contiguous(), delta.to(hidden.dtype).contiguous(), base.to(hidden.dtype).contiguous()
    r = None if residual is None else residual.to(hidden.dtype).contiguous()
    out = torch.empty_like(h)
    _check(lib().telb_dflash2_conv(_p(h), _p(d), _p(b), _p(r), _p(out), c_int(h.shape[0]), c_int(h.shape[1]), c_int(block),
                                   c_int(b.shape[0]), c_int(group_size), c_int(int(h.dtype == torch.bfloat16)), _stream()), "dflash2_conv")
    return out


def dflash2_selector_walk(cand_ids, unary, projected, anchor, pred_codebook, succ_codebook, temperatures=None, uniforms=None):
    """DFlash 2's chain selector: ``(tokens [B, S] int64, probabilities [B, S, K] fp32)``."""
    assert projected.dtype in (torch.float16, torch.bfloat16) and pred_codebook.dtype == projected.dtype == succ_codebook.dtype
    b, s, k = cand_ids.shape
    dev = cand_ids.device
    c, u, z = cand_ids.to(torch.int32).contiguous(), unary.float().contiguous(), projected.contiguous()
    a, pc, qc = anchor.to(device=dev, dtype=torch.int32).contiguous(), pred_codebook.contiguous(), succ_codebook.contiguous()
    t = None if temperatures is None else temperatures.to(device=dev, dtype=torch.float32).contiguous()
    un = None if uniforms is None else uniforms.to(device=dev, dtype=torch.float32).contiguous()
    tok = torch.empty(b, s, dtype=torch.int32, device=dev)
    pr = torch.empty(b, s, k, dtype=torch.float32, device=dev)
    _check(lib().telb_dflash2_selector(_p(c), _p(u), _p(z), _p(a), _p(pc), _p(qc), _p(t), _p(un), _p(tok), _p(pr), c_int(b), c_int(s), c_int(k),
                                       c_int(z.shape[-1]), c_int(pc.shape[0]), c_int(int(z.dtype == torch.bfloat16)), _stream()),
           "dflash2_selector")
    return tok.long(), pr


def spec_accept_sampling(target_probs, tree_tokens, parents, max_path: int, uniforms):
    """Lossless tree acceptance of sampled requests on the device: ``(path [B, max_path], path_len [B], bonus [B])`` int32."""
    b, n, v = target_probs.shape
    dev = target_probs.device
    pr = target_probs.float().contiguous()
    tok, par = tree_tokens.to(device=dev, dtype=torch.int32).contiguous(), parents.to(device=dev, dtype=torch.int32).contiguous()
    u = uniforms.to(device=dev, dtype=torch.float32).contiguous()
    assert u.shape[0] == b and u.shape[1] >= max_path and u.shape[2] >= 2
    if u.shape[1] != max_path:
        u = u[:, :max_path].contiguous()
    path = torch.empty(b, max_path, dtype=torch.int32, device=dev)
    plen = torch.empty(b, dtype=torch.int32, device=dev)
    bonus = torch.empty(b, dtype=torch.int32, device=dev)
    _check(lib().telb_spec_accept_sampling(_p(pr), _p(tok), _p(par), _p(u), _p(path), _p(plen), _p(bonus), c_int(b), c_int(n), c_int(v),
                                           c_int(max_path), c_int(u.shape[2]), _stream()), "spec_accept_sampling")
    return path, plen, bonus


def markov_greedy_chain(logits, w1, w2, first_prev):
    """Greedy chain of DSpark's Markov head over ``logits [B, P, V]`` (fp32): ``P`` fused correction + arg-max launches."""
    assert w1.dtype == w2.dtype and w1.dtype in (torch.float16, torch.bfloat16) and w1.shape[1] == w2.shape[1]
    b, p, v = logits.shape
    lg, a, c = logits.float().contiguous(), w1.contiguous(), w2.contiguous()
    fp = first_prev.to(device=lg.device, dtype=torch.int32).contiguous()
    slots = torch.empty(b * p, dtype=torch.int64, device=lg.device)
    tok = torch.empty(b, p, dtype=torch.int32, device=lg.device)
    _check(lib().telb_markov_greedy_chain(_p(lg), _p(a), _p(c), _p(fp), _p(slots), _p(tok), c_int(b), c_int(p), c_int(v), c_int(a.shape[0]),
                                          c_int(a.shape[1]), c_int(int(a.dtype == torch.bfloat16)), _stream()), "markov_greedy_chain")
    return tok.long()


def lattice_chain_walk(cand_ids, transition, temperatures=None, uniforms=None):
    """Walk of a candidate lattice with per-slot ``[prev, next]`` transition scores: ``(tokens [B, S] int64, probabilities)``."""
    b, s, k = cand_ids.shape
    dev = cand_ids.device
    c, tr = cand_ids.to(torch.int32).contiguous(), transition.float().contiguous()
    t = None if temperatures is None else temperatures.to(device=dev, dtype=torch.float32).contiguous()
    un = None if uniforms is None else uniforms.to(device=dev, dtype=torch.float32).contiguous()
    tok = torch.empty(b, s, dtype=torch.int32, device=dev)
    pr = torch.empty(b, s, k, dtype=torch.float32, device=dev)
    _check(lib().telb_lattice_chain_walk(_p(c), _p(tr), _p(t), _p(un), _p(tok), _p(pr), c_int(b), c_int(s), c_int(k), _stream()),
           "lattice_chain_walk")
    return tok.long(), pr


def candidate_rescore(hidden, lm_head, cand):
    """Exact logits of each row's candidate tokens, ordered (logit descending, id ascending), with the log-softmax over the set:
    ``(ids [R, Kc] int32, log-probabilities [R, Kc] fp32)``."""
    assert hidden.dtype == lm_head.dtype and hidden.dtype in (torch.float16, torch.bfloat16)
    h, w, c = hidden.contiguous(), lm_head.contiguous(), cand.to(torch.int32).contiguous()
    rows, kc = c.shape
    ids = torch.empty(rows, kc, dtype=torch.int32, device=h.device)
    lp = torch.empty(rows, kc, dtype=torch.float32, device=h.device)
    _check(lib().telb_candidate_rescore(_p(h), _p(w), _p(c), _p(ids), _p(lp), c_int(rows), c_int(h.shape[1]), c_int(kc),
                                        c_int(w.shape[0]), c_int(int(h.dtype == torch.bfloat16)), _stream()), "candidate_rescore")
    return ids, lp


def kv_commit_path(pool, page_table, past_len, path, path_len) -> None:
    assert pool.is_contiguous() and pool.element_size() in (1, 2)
    if pool.element_size() == 1:            # FP8 pages: a row of D bytes moves as D / 2 16-bit elements
        pool = pool.view(torch.int16)
    layers, pages, _, hkv, psz, d = pool.shape
    pt, pl, pth, pln = page_table.to(torch.int32).contiguous(), past_len.to(torch.int32).contiguous(), path.contiguous(), path_len.contiguous()
    _check(lib().telb_kv_commit_path(_p(pool), _p(pt), _p(pl), _p(pth), _p(pln), c_int(path.shape[0]), c_int(path.shape[1]),
                                     c_int(page_table.shape[1]), c_int(layers), c_int(pages), c_int(hkv), c_int(psz), c_int(d),
                                     _stream()), "kv_commit_path")
