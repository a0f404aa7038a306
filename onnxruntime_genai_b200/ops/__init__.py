"""Device ops.  CUDA tensors run the hand-written sm_100a kernels (ctypes into
libogb200_kernels.so); CPU tensors run the fp32 PyTorch restatements in `reference.py`.

There is deliberately no third path: a CUDA tensor never falls back to PyTorch math, and a missing
kernel library on a GPU machine is an error.
"""
from __future__ import annotations

import math
import os
from typing import Optional, Tuple

import numpy as np
import torch

from . import reference as ref
from . import _lib
from .fp4 import Fp4Experts
from .w4 import QuantizedEmbedding, W4Weight, unpack_ort_q4

_ACT = {"silu": 0, "gelu": 1, "gelu_tanh": 1, "relu": 2, "gelu_erf": 3, "relu2": 4}


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def _stream():
    return torch.cuda.current_stream().cuda_stream


class _Workspace:
    """Per-device state shared by the kernels: the status word and the split-KV scratch of attention
    (the GEMM's split-K reduces on chip and needs none).  Allocated once (outside graph capture)."""

    def __init__(self, device: torch.device):
        self.device = device
        idx = device.index if device.index is not None else torch.cuda.current_device()
        self.index = idx
        _lib.init_device(idx)
        self.status = _lib.lib().ogb_status_device_ptr(idx)
        self.sm_count = _lib.lib().ogb_sm_count(idx)
        self.attn_ws = torch.empty(64 << 20, dtype=torch.uint8, device=device)
        self._retired = []

    def attn_scratch(self, nbytes: int) -> torch.Tensor:
        if nbytes > self.attn_ws.numel():
            if torch.cuda.is_current_stream_capturing():
                raise RuntimeError("attention scratch too small during CUDA graph capture; warm up eagerly first")
            # captured graphs hold the raw address of the buffer they were recorded with: a replaced buffer is kept alive
            # for the life of the process instead of going back to the allocator, where a replay would write into it
            self._retired.append(self.attn_ws)
            self.attn_ws = torch.empty(int(nbytes * 1.25), dtype=torch.uint8, device=self.device)
        return self.attn_ws


_workspaces = {}


def workspace(device: torch.device) -> _Workspace:
    key = device.index if device.index is not None else torch.cuda.current_device()
    ws = _workspaces.get(key)
    if ws is None:
        ws = _workspaces[key] = _Workspace(torch.device("cuda", key))
    return ws


def check_kernel_status(device=None) -> None:
    """Synchronises and raises if any kernel reported that a bounded wait ran out."""
    idx = torch.cuda.current_device() if device is None else torch.device(device).index
    _lib.init_device(idx)
    _lib.check_status(idx)


# ------------------------------------------------------------------------------------------ graph capture
import contextlib
import gc


@contextlib.contextmanager
def graph_capture(graph, **kw):
    """torch.cuda.graph with the cyclic garbage collector off for the duration of the capture: a collected object that owns CUDA
    resources (an older graph, a pinned buffer) frees them from inside the capture and invalidates it
    ("operation failed due to a previous error during capture" at the next launch)."""
    was_on = gc.isenabled()
    gc.disable()
    try:
        with torch.cuda.graph(graph, **kw):
            yield
    finally:
        if was_on:
            gc.enable()


# ------------------------------------------------------------------------------------------ debug bounds checks
# OGB_DEBUG_BOUNDS=1: every index tensor an op is about to hand to a kernel (token ids, cache slots, block-table entries,
# gathered rows, rotary positions) is range-checked first and a bad one raises IndexError naming the op, instead of the kernel
# reading or writing out of bounds.  The checks synchronise the stream, so this is a debugging mode (and CUDA graphs that
# were captured with it on replay without checks).
DEBUG_BOUNDS = os.environ.get("OGB_DEBUG_BOUNDS", "0") == "1"


def _check_index(op: str, name: str, t, hi: int, lo: int = 0) -> None:
    if not DEBUG_BOUNDS or t is None or t.numel() == 0 or (t.is_cuda and torch.cuda.is_current_stream_capturing()):
        return
    bad = (t < lo) | (t >= hi)
    if bool(bad.any()):
        v = t[bad].flatten()[0].item()
        raise IndexError(f"{op}: {name} holds {v}, outside [{lo}, {hi})")


# ------------------------------------------------------------------------------------------ embedding
def embedding(ids: torch.Tensor, table, scale: float = 1.0) -> torch.Tensor:
    _check_index("embedding", "ids", ids, table.V if isinstance(table, QuantizedEmbedding) else table.shape[0])
    if isinstance(table, QuantizedEmbedding):
        if table.device.type != "cuda":
            return ref.embedding(ids, table.dequantize(), scale)
        T = ids.numel()
        out = torch.empty(T, table.K, dtype=torch.bfloat16, device=table.device)
        _lib.check(_lib.lib().ogb_embedding_q4(_ptr(ids), _ptr(table.q), _ptr(table.scales), _ptr(table.zp), _ptr(out), T, table.K,
                                              table.V, float(scale), _stream()), "embedding_q4")
        return out
    if not table.is_cuda:
        return ref.embedding(ids, table, scale)
    assert table.dtype == torch.bfloat16 and ids.dtype == torch.int32
    T, H = ids.numel(), table.shape[1]
    out = torch.empty(T, H, dtype=table.dtype, device=table.device)
    _lib.check(_lib.lib().ogb_embedding(_ptr(ids), _ptr(table), _ptr(out), T, H, table.shape[0], float(scale), _stream()), "embedding")
    return out


def embedding_stream(ids: torch.Tensor, table: torch.Tensor, scale: float = 1.0, dtype=None):
    """Embedding rows as the start of an fp32 residual stream (bf16 or fp32 table, any width).  With `dtype`: (stream, the rows in that
    type), the stream itself where it is fp32."""
    _check_index("embedding_stream", "ids", ids, table.shape[0])
    if not table.is_cuda:
        h = ref.embedding(ids, table).float() * scale
        return h if dtype is None else (h, h if dtype == torch.float32 else h.to(dtype))
    assert ids.dtype == torch.int32 and table.is_contiguous() and table.dtype in (torch.bfloat16, torch.float32)
    T, H = ids.numel(), table.shape[1]
    out = torch.empty(T, H, dtype=torch.float32, device=table.device)
    copy = torch.empty(T, H, dtype=torch.bfloat16, device=table.device) if dtype == torch.bfloat16 else None
    _lib.check(_lib.lib().ogb_embedding_stream(_ptr(ids), _ptr(table), int(table.dtype == torch.float32), _ptr(out), _ptr(copy), T, H, table.shape[0],
                                              float(scale), _stream()), "embedding_stream")
    return out if dtype is None else (out, out if copy is None else copy)


def add_normed(h, y, weight, eps, dtype=torch.bfloat16):
    """h += weight * v / rms(v) in place: the normed output of a sub-layer joins the fp32 residual stream h [T, H].  v = y [T, H], or the
    weighted sum of a mixture-of-experts layer whose combine step is pending.  weight fp32 [H].  Returns the new stream in `dtype` (the
    stream itself where that is fp32)."""
    if not h.is_cuda:
        ref.add_normed(h, y, weight, eps)
        return h if dtype == torch.float32 else h.to(dtype)
    plan = None
    if isinstance(y, PendingCombine):
        assert y.shared is None
        y, plan = y.y, y.plan
    T, H = h.shape
    assert h.dtype == torch.float32 and h.is_contiguous() and weight.dtype == torch.float32 and y.stride(1) == 1 and y.shape[1] == H
    assert y.dtype in (torch.bfloat16, torch.float32) and (plan is None or plan.T == T)
    x = torch.empty(T, H, dtype=torch.bfloat16, device=h.device) if dtype == torch.bfloat16 else None
    _lib.check(_lib.lib().ogb_add_normed(_ptr(h), _ptr(y), y.stride(0), int(y.dtype == torch.float32), _ptr(weight), float(eps), _ptr(x),
                                        _ptr(plan.inv_pos) if plan else None, _ptr(plan.topk_w) if plan else None, plan.k if plan else 0, T, H, _stream()),
               "add_normed")
    return h if x is None else x


def embedding_bigram(ids, table, scale, bigram, spec, tokens, slots, positions, cu_seqlens, past_lens, block_table, block_size: int):
    """Start of an fp32 residual stream: table[id] * scale + bigram[(previous * mul_prev + id * mul_cur) mod buckets] (row `buckets` for the first
    token of a sequence), spec = {buckets, mul_prev, mul_cur}.  The token before a request's first one of the step is read from the paged pool
    `tokens` [slots] int32, to which this step's tokens are written (slot < 0: not)."""
    _check_index("embedding_bigram", "slots", slots[:ids.numel()], tokens.shape[0], -1)
    if not table.is_cuda:
        return ref.embedding_bigram(ids, table, scale, bigram, spec, tokens, slots, positions, cu_seqlens, past_lens, block_table, block_size)
    import ctypes
    assert ids.dtype == torch.int32 and tokens.dtype == torch.int32 and table.is_contiguous() and bigram.is_contiguous() and bigram.dtype == table.dtype
    assert bigram.shape == (spec["buckets"] + 1, table.shape[1]) and block_table.stride(1) == 1 and table.dtype in (torch.bfloat16, torch.float32)
    T, H = ids.numel(), table.shape[1]
    out = torch.empty(T, H, dtype=torch.float32, device=table.device)
    p = _lib.Bigram(ids=_ptr(ids), slots=_ptr(slots), positions=_ptr(positions), cu_seqlens=_ptr(cu_seqlens), block_table=_ptr(block_table),
                    tokens=_ptr(tokens), table_cols=block_table.stride(0), block_size=int(block_size), B=past_lens.shape[0], T=T, H=H, vocab=table.shape[0],
                    fp32=int(table.dtype == torch.float32), scale=float(scale), **spec)
    _lib.check(_lib.lib().ogb_embedding_bigram(ctypes.byref(p), _ptr(table), _ptr(bigram), _ptr(out), _stream()), "embedding_bigram")
    return out


class TanhNorm:
    """A norm without statistics: tanh(alpha * x) * weight + bias (weight and bias fp32)."""
    __slots__ = ("weight", "bias", "alpha")

    def __init__(self, weight, bias, alpha: float):
        self.weight, self.bias, self.alpha = weight, bias, float(alpha)


def add_tanh_norm(h, y, norm: TanhNorm, dtype=torch.bfloat16, first=None, step=None, rows=None, out=None):
    """n = h + y (+ first) (+ step), tanh norm of n in `dtype`; n is written to `out` (h itself: in place; None: nowhere).  h [T, H] the fp32 residual
    stream; y: the sub-layer's rows [T, H], a mixture-of-experts output whose combine step is pending, or None; first fp32 [T, H], step fp32 [H].
    rows (int32): only these rows are summed and normed (out must be None)."""
    if not h.is_cuda:
        return ref.add_tanh_norm(h, y, norm, dtype, first, step, rows, out)
    import ctypes
    plan = y2 = None
    if isinstance(y, PendingCombine):
        y, plan, y2 = y.y, y.plan, y.shared
    T, H = h.shape
    n = T if rows is None else rows.numel()
    assert h.dtype == torch.float32 and h.is_contiguous() and (out is None or (rows is None and out.is_contiguous() and out.dtype == torch.float32))
    assert all(t is None or (t.dtype == dtype and t.stride(1) == 1 and t.shape[1] == H) for t in (y, y2)) and norm.weight.dtype == torch.float32
    assert all(t is None or (t.dtype == torch.float32 and t.is_contiguous()) for t in (first, step)) and (plan is None or plan.T == T)
    x = torch.empty(n, H, dtype=dtype, device=h.device)
    p = _lib.TanhNorm(h_in=_ptr(h), h_out=_ptr(out), y=_ptr(y), y2=_ptr(y2), inv_pos=_ptr(plan.inv_pos) if plan else None,
                      topk_w=_ptr(plan.topk_w) if plan else None, first=_ptr(first), step=_ptr(step), w=_ptr(norm.weight), b=_ptr(norm.bias), x=_ptr(x),
                      rows=_ptr(rows), ldy=y.stride(0) if y is not None else 0, ldy2=y2.stride(0) if y2 is not None else 0, k=plan.k if plan else 0,
                      n_rows=n, H=H, fp32=int(dtype == torch.float32), alpha=norm.alpha)
    _lib.check(_lib.lib().ogb_add_tanh_norm(ctypes.byref(p), _stream()), "add_tanh_norm")
    return x


def norm_stream(x, weight, eps, bias=None, layernorm=False, dtype=torch.bfloat16, rows=None, add=None, weight2=None):
    """Norm of the rows of an fp32 residual stream [T, H] (of the rows listed in `rows`, int32, when given) as `dtype`; weight and bias
    are fp32.  add: rows [T, H] in `dtype`, or a mixture-of-experts output whose combine step is pending, that join the stream first (in place,
    where all its rows are normed).  weight2: returns the pair (norm with weight and bias, norm with weight2)."""
    if rows is not None:
        _check_index("norm_stream", "rows", rows, x.shape[0])
    if not x.is_cuda:
        if add is not None:
            x = x.add_(add.float()) if rows is None else x + add.float()
        h = x if rows is None else x[rows.long()]
        one = lambda w, b: ref.norm(h.float(), w, eps, None, b, layernorm)[0].to(dtype)
        return one(weight, bias) if weight2 is None else (one(weight, bias), one(weight2, None))
    import ctypes
    plan = None
    if isinstance(add, PendingCombine):
        assert add.shared is None
        add, plan = add.y, add.plan
    assert x.dtype == torch.float32 and x.is_contiguous() and all(t is None or t.dtype == torch.float32 for t in (weight, bias, weight2))
    n, H = (x.shape[0] if rows is None else rows.numel()), x.shape[1]
    assert add is None or (add.dtype == dtype and add.stride(1) == 1 and add.shape[1] == H) and (plan is None or plan.T == x.shape[0])
    out = torch.empty(n, H, dtype=dtype, device=x.device)
    out2 = torch.empty_like(out) if weight2 is not None else None
    p = _lib.NormStream(x=_ptr(x), rows=_ptr(rows), w=_ptr(weight), b=_ptr(bias), w2=_ptr(weight2), out=_ptr(out), out2=_ptr(out2), y=_ptr(add),
                        inv_pos=_ptr(plan.inv_pos) if plan else None, topk_w=_ptr(plan.topk_w) if plan else None, ldy=add.stride(0) if add is not None else 0,
                        k=plan.k if plan else 0, n_rows=n, H=H, layernorm=int(layernorm), fp32=int(dtype == torch.float32), eps=float(eps))
    _lib.check(_lib.lib().ogb_norm_stream(ctypes.byref(p), _stream()), "norm_stream")
    return out if out2 is None else (out, out2)


# ------------------------------------------------------------------------------------------ norm
def norm(x, weight, eps, residual=None, bias=None, layernorm=False, out=None) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """Returns (normalised, new_residual).  With `residual`, normalises x + residual and returns the
    sum as new_residual (written in place into `residual`)."""
    if not x.is_cuda:
        y, r = ref.norm(x, weight, eps, residual, bias, layernorm)
        if residual is not None:
            residual.copy_(r)
            r = residual
        return y, r
    assert x.dtype == torch.bfloat16 and x.is_contiguous()
    rows, H = x.shape
    if out is None:
        out = torch.empty_like(x)
    _lib.check(_lib.lib().ogb_norm(_ptr(x), _ptr(residual), _ptr(residual), _ptr(weight), _ptr(bias), _ptr(out), rows, H,
                                   float(eps), int(layernorm), _stream()), "norm")
    return out, residual


class PendingCombine:
    """The output of a mixture-of-experts layer before its combine step: the experts' rows `y` and the routing plan.
    `norm_moe_combine` folds the weighted sum into the residual add + norm that consumes it.  shared: rows [T, H] of an expert that runs for
    every token outside the routing plan (added with weight 1)."""
    __slots__ = ("y", "plan", "shared")

    def __init__(self, y, plan, shared=None):
        self.y, self.plan, self.shared = y, plan, shared


def norm_moe_combine(pending: PendingCombine, weight, eps, residual, bias=None, layernorm=False):
    """norm(moe_combine(pending.y, pending.plan), weight, eps, residual, ...) in one launch; same results bit for bit."""
    y, plan = pending.y, pending.plan
    assert pending.shared is None and y.is_cuda and y.dtype == torch.bfloat16 and y.stride(-1) == 1 and residual is not None
    H = y.shape[1]
    out = torch.empty(plan.T, H, dtype=torch.bfloat16, device=y.device)
    _lib.check(_lib.lib().ogb_norm_moe_combine(_ptr(y), y.stride(0), _ptr(plan.inv_pos), _ptr(plan.topk_w), plan.k, _ptr(residual),
                                               _ptr(residual), _ptr(weight), _ptr(bias), _ptr(out), plan.T, H, float(eps), int(layernorm),
                                               _stream()), "norm_moe_combine")
    return out, residual


# ------------------------------------------------------------------------------------------ GEMM
GEMM_FP32_OUT, GEMM_ACT_PAIR, GEMM_ALLREDUCE, GEMM_REDUCE_SCATTER, GEMM_GATHERED_A, GEMM_FP32_RESIDUAL, GEMM_PAIR_RELU, GEMM_PAIR_GELU = 1, 2, 4, 8, 16, 32, 64, 128


FUSED_MAX_TOKENS = 128     # the decode-step fusions (folded norm, rotary + cache append) run in the decode-sized GEMM kernel


def _gemm(x, w, out, bias, residual, flags, splits, fused=None):
    ws = workspace(x.device)
    T, K = x.shape
    if fused is None:
        rc = _lib.lib().ogb_gemm_bf16(_ptr(x), x.stride(0), _ptr(w), w.stride(0), _ptr(out), out.stride(0), T, w.shape[0], K, _ptr(bias),
                                      _ptr(residual), residual.stride(0) if residual is not None else 0, int(flags), int(splits),
                                      ws.index, ws.status, ws.sm_count, _stream())
    else:
        import ctypes
        rc = _lib.lib().ogb_gemm_bf16_fused(_ptr(x), x.stride(0), _ptr(w), w.stride(0), _ptr(out), out.stride(0), T, w.shape[0], K,
                                            _ptr(bias), _ptr(residual), residual.stride(0) if residual is not None else 0, int(flags),
                                            int(splits), ws.index, ws.status, ws.sm_count, _stream(), ctypes.byref(fused))
    _lib.check(rc, "gemm_bf16")
    return out


_ones = {}


def _unit_weight(n: int, device) -> torch.Tensor:
    key = (n, str(device))
    t = _ones.get(key)
    if t is None:
        t = _ones[key] = torch.ones(n, dtype=torch.bfloat16, device=device)
    return t


def rms_scale(x, eps: float):
    """x / rms(x) (no weight): the rows a GEMM with a folded norm would see, for the paths that cannot fold."""
    if not x.is_cuda:
        return ref.rms_scale(x, eps)
    return norm(x, _unit_weight(x.shape[1], x.device), eps)[0]


def _gemm_w4(x, w, out, bias, residual, flags, splits):
    ws = workspace(x.device)
    rc = _lib.lib().ogb_gemm_w4(_ptr(x), x.stride(0), _ptr(w.packed), _ptr(out), out.stride(0), x.shape[0], w.N, w.K, _ptr(bias),
                                _ptr(residual), residual.stride(0) if residual is not None else 0, int(flags), int(splits),
                                ws.status, ws.sm_count, _stream())
    _lib.check(rc, "gemm_w4")
    return out


def _tma_ok(x, w) -> bool:
    """TMA can address both operands of a bf16 product: 16-byte row strides and addresses."""
    return x.shape[1] % 8 == 0 and x.stride(0) % 8 == 0 and w.stride(0) % 8 == 0 and (x.data_ptr() | w.data_ptr()) % 16 == 0


def _gemm_simt(x, w, out, residual=None, batch=1, a_cols=0, c_cols=0, K=None, bias=None, act=0):
    """The fp32 / unaligned form of a product (csrc/gemm_simt.cu)."""
    assert bias is None or bias.dtype == x.dtype
    assert x.dtype == w.dtype and x.dtype in (torch.float32, torch.bfloat16) and out.dtype in (torch.float32, torch.bfloat16)
    _lib.check(_lib.lib().ogb_gemm_simt(_ptr(x), x.stride(0), int(a_cols), _ptr(w), w.stride(0), _ptr(out), out.stride(0), int(c_cols), x.shape[0],
                                       w.shape[0] // batch, K or x.shape[1], int(batch), _ptr(residual), residual.stride(0) if residual is not None else 0,
                                       _ptr(bias), int(act), int(x.dtype == torch.float32), int(out.dtype == torch.float32), _stream()), "gemm_simt")
    return out


def head_project(x, w, heads: int, a_cols: int, out=None, gate=None):
    """Per-head products over the same token rows: out[:, h * N + n] = sum_k x[:, h * a_cols + k] * w[h * N + n, k] with
    w [heads * N, K]; x may be wider than the heads need; gate [T, heads * N]: the result is multiplied by its sigmoid.  Returns [T, heads * N] (or
    writes `out`, which may be a column range)."""
    K, N = w.shape[1], w.shape[0] // heads
    if out is None:
        out = torch.empty(x.shape[0], heads * N, dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        out.copy_(ref.head_project(x, w, heads, a_cols))
        return out if gate is None else gate_rows(out, gate)
    if x.dtype == torch.float32 or a_cols % 8 or K % 8 or x.stride(0) % 8 or w.stride(0) % 8 or (x.data_ptr() | w.data_ptr()) % 16:
        _gemm_simt(x, w, out, batch=heads, a_cols=a_cols, c_cols=N, K=K)
        return out if gate is None else gate_rows(out, gate)
    assert x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and out.dtype == torch.bfloat16
    assert gate is None or (gate.dtype == torch.bfloat16 and gate.stride(1) == 1 and gate.shape == (x.shape[0], heads * N))
    _lib.check(_lib.lib().ogb_gemm_bf16_batched(_ptr(x), x.stride(0), x.shape[1], int(a_cols), _ptr(w), w.stride(0), _ptr(out), out.stride(0), N,
                                               x.shape[0], N, K, heads, _ptr(gate), gate.stride(0) if gate is not None else 0,
                                               workspace(x.device).status, _stream()), "gemm_bf16_batched")
    return out


def linear(x, w, bias=None, residual=None, out_fp32=False, out=None, splits=0, all_reduce=False, reduce_scatter=None, norm_eps=0.0):
    """y = x @ w.T (+bias) (+residual).  x [T, K] bf16, w [N, K] bf16 (K contiguous).  With all_reduce the
    partial products of the tensor-parallel ranks are summed inside the kernel over NVLink peer memory.
    reduce_scatter=(rank, world): the sum is scattered by token rows instead (sequence-parallel form): the result has
    this rank's rows [rank * ceil(T / world), ...) only, and `residual` is that slice.
    norm_eps > 0: an RMS norm folded into the GEMM - x holds the un-normalised rows, w already carries the norm's weight
    (w * norm_weight along K), and row m of the product is scaled by rsqrt(mean(x[m]^2) + norm_eps)."""
    if isinstance(w, W4Weight):
        if norm_eps > 0:
            x = rms_scale(x, norm_eps)
        if not x.is_cuda:
            return ref.linear(x, w.dequantize(), bias, residual, out_fp32)
        if all_reduce:
            raise RuntimeError("the fused all-reduce is not available for int4 weights")
        if out is None:
            out = torch.empty(x.shape[0], w.N, dtype=torch.float32 if out_fp32 else torch.bfloat16, device=x.device)
        return _gemm_w4(x, w, out, bias, residual, GEMM_FP32_OUT if out_fp32 else 0, splits)
    if not x.is_cuda:
        y = ref.linear(x, w, bias, residual, out_fp32, norm_eps)
        return y if out is None else out.copy_(y)
    assert x.dtype == w.dtype and x.stride(-1) == 1 and w.stride(-1) == 1
    if x.dtype == torch.float32 or (norm_eps == 0 and not all_reduce and reduce_scatter is None and not _tma_ok(x, w) and
                                    (residual is None or residual.dtype == torch.float32)):
        # 32-bit models, and bf16 shapes TMA cannot address
        assert norm_eps == 0 and not all_reduce and reduce_scatter is None
        if out is None:
            out = torch.empty(x.shape[0], w.shape[0], dtype=torch.float32 if out_fp32 else x.dtype, device=x.device)
        return _gemm_simt(x, w, out, residual, bias=bias)
    assert x.dtype == torch.bfloat16
    fused = None
    if norm_eps > 0:
        if x.shape[0] > FUSED_MAX_TOKENS:
            x = rms_scale(x, norm_eps)     # prefill-sized steps run the persistent kernel: normalise first
        else:
            fused = _lib.GemmFused(norm_eps=float(norm_eps))
    rows_out = x.shape[0]
    if reduce_scatter is not None:
        rank, world = reduce_scatter
        per = -(-x.shape[0] // world)
        rows_out = max(0, min(per, x.shape[0] - rank * per))
    if out is None:
        out = torch.empty(rows_out, w.shape[0], dtype=torch.float32 if out_fp32 else torch.bfloat16, device=x.device)
    flags = (GEMM_FP32_OUT if out_fp32 else 0) | (GEMM_ALLREDUCE if all_reduce else 0) | (GEMM_REDUCE_SCATTER if reduce_scatter else 0)
    if residual is not None and residual.dtype == torch.float32:
        flags |= GEMM_FP32_RESIDUAL       # an fp32 residual stream, updated in place by the epilogue when `out` is the residual itself
    return _gemm(x, w, out, bias, residual, flags, splits, fused)


def linear_act(x, w, act, out=None):
    """act(x @ w.T), the activation in the product's epilogue; `out` may be a column range of a wider matrix."""
    if not x.is_cuda:
        y = ref.linear_act(x, w, act)
        return y if out is None else out.copy_(y)
    if out is None:
        out = torch.empty(x.shape[0], w.shape[0], dtype=x.dtype, device=x.device)
    assert x.dtype == w.dtype == out.dtype and x.stride(1) == 1 and w.stride(1) == 1 and out.stride(1) == 1
    if x.dtype == torch.float32 or not _tma_ok(x, w):
        return _gemm_simt(x, w, out, act=1 + _ACT[act])
    return _gemm(x, w, out, None, None, (1 + _ACT[act]) << 8, 0)


def qkv_rope_append(x, w, bias, positions, slots, cos_cache, sin_cache, k_cache, v_cache, Hq, Hkv, D, rot, norm_eps=0.0):
    """QKV projection + rotary embedding + KV-cache append (+ folded RMS norm) as one kernel for decode-sized steps.
    Returns a tensor whose first Hq * D columns are the rotated queries (what paged_attention reads); rotated keys and the
    values of token m are written to row slots[m] of the caches.  Non-interleaved rotation only; head_dim must divide 128,
    the rotary dimension must be a multiple of 16 and the caches bf16 - `qkv_fusable` tells; other cases (and prefill-sized
    steps) take the separate kernels."""
    T = x.shape[0]
    _check_index("qkv_rope_append", "slots", slots[:T], k_cache.shape[0], -1)
    if cos_cache is not None:
        _check_index("qkv_rope_append", "positions", positions[:T], cos_cache.shape[0])
    if x.is_cuda and T <= FUSED_MAX_TOKENS and not isinstance(w, W4Weight) and qkv_fusable(D, rot, k_cache):
        assert x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.shape[0] == (Hq + 2 * Hkv) * D
        q = torch.empty(T, Hq * D, dtype=torch.bfloat16, device=x.device)
        f = _lib.GemmFused(norm_eps=float(norm_eps), positions=_ptr(positions), slots=_ptr(slots), cos=_ptr(cos_cache), sin=_ptr(sin_cache),
                           k_cache=_ptr(k_cache), v_cache=_ptr(v_cache), Hq=Hq, Hkv=Hkv, D=D, rot=int(rot if cos_cache is not None else 0),
                           max_pos=cos_cache.shape[0] if cos_cache is not None else 1)
        return _gemm(x, w, q, bias, None, 0, 0, f)
    qkv = linear(x, w, bias, norm_eps=norm_eps)
    rope_kv_append(qkv, positions, slots, cos_cache, sin_cache, k_cache, v_cache, Hq, Hkv, D, rot)
    return qkv


def qkv_fusable(D: int, rot: int, k_cache) -> bool:
    return 128 % D == 0 and rot % 16 == 0 and k_cache.dtype == torch.bfloat16


def linear_gathered(M: int, w, bias=None, out_fp32=False, act_pair=False, splits=0):
    """all-gather -> GEMM in one kernel: y[M, N] = X @ w.T where X's token rows were pushed by the ranks with
    `comm.all_gather_push` (rank r: rows [r * ceil(M / world), ...)) just before; the kernel builds its activation
    tiles from the flagged lines in the local receive buffer as they arrive.  act_pair: silu(gate) * up epilogue for
    weights in the 64-row gate/up block layout."""
    N, K = w.shape
    dev = w.device
    out = torch.empty(M, N // 2 if act_pair else N, dtype=torch.float32 if out_fp32 else torch.bfloat16, device=dev)
    ws = workspace(dev)
    flags = (GEMM_FP32_OUT if out_fp32 else 0) | (GEMM_ACT_PAIR if act_pair else 0) | GEMM_GATHERED_A
    rc = _lib.lib().ogb_gemm_bf16(_ptr(w), K, _ptr(w), w.stride(0), _ptr(out), out.stride(0), M, N, K, _ptr(bias), None, 0, int(flags),
                                  int(splits), ws.index, ws.status, ws.sm_count, _stream())
    _lib.check(rc, "gemm_bf16 (gathered activations)")
    return out


def interleave_gate_up(w: torch.Tensor, block: int = 64) -> torch.Tensor:
    """[gate; up] stacked rows ([2I, ...]) -> blocks of 64 gate rows followed by the 64 up rows of the same
    features, the row order the paired-activation GEMM epilogue expects.  Works for weights and biases."""
    inter = w.shape[0] // 2
    assert inter % block == 0
    g, u = w[:inter].reshape(inter // block, 1, block, *w.shape[1:]), w[inter:].reshape(inter // block, 1, block, *w.shape[1:])
    return torch.cat([g, u], dim=1).reshape(w.shape).contiguous()


_PAIR_FLAGS = {"silu": 0, "relu": GEMM_PAIR_RELU, "gelu_tanh": GEMM_PAIR_GELU, "gelu": GEMM_PAIR_GELU}      # activations the GEMM's epilogue pairs


def gate_up_act(x, w, bias=None, act="silu", out=None, splits=0, interleaved=False, norm_eps=0.0):
    """act(x @ Wg.T) * (x @ Wu.T).  w is [2I, K]: stacked [Wg; Wu], or (interleaved=True) blocks of 64 gate
    rows + 64 up rows as produced by interleave_gate_up (the layout the fused kernel needs).  norm_eps: as in `linear`."""
    fused = None
    if norm_eps > 0:
        if not x.is_cuda:
            return ref.gate_up_act(x, w.dequantize() if isinstance(w, W4Weight) else w, bias, act,
                                   w.interleaved if isinstance(w, W4Weight) else interleaved, norm_eps)
        if isinstance(w, W4Weight) or x.shape[0] > FUSED_MAX_TOKENS or act != "silu" or not interleaved or (w.shape[0] // 2) % 64:
            x = rms_scale(x, norm_eps)
        else:
            fused = _lib.GemmFused(norm_eps=float(norm_eps))
    if isinstance(w, W4Weight):
        if not x.is_cuda:
            return ref.gate_up_act(x, w.dequantize(), bias, act, w.interleaved)
        inter = w.N // 2
        if act == "silu" and w.interleaved:
            if out is None:
                out = torch.empty(x.shape[0], inter, dtype=torch.bfloat16, device=x.device)
            return _gemm_w4(x, w, out, bias, None, GEMM_ACT_PAIR, splits)
        y = linear(x, w, bias)
        if w.interleaved:
            y = y.view(-1, inter // 64, 2, 64).transpose(1, 2).reshape(-1, 2 * inter)
        return act_mul(y.contiguous(), act)
    if not x.is_cuda:
        y = ref.gate_up_act(x, w, bias, act, interleaved)
        return y if out is None else out.copy_(y)
    inter = w.shape[0] // 2
    if act not in _PAIR_FLAGS or not interleaved or inter % 64 or x.dtype != torch.bfloat16 or not _tma_ok(x, w):
        y = linear(x, w, bias)
        if interleaved:
            y = y.view(-1, inter // 64, 2, 64).transpose(1, 2).reshape(-1, 2 * inter)
        return act_mul(y.contiguous(), act, out)
    if out is None:
        out = torch.empty(x.shape[0], inter, dtype=torch.bfloat16, device=x.device)
    return _gemm(x, w, out, bias, None, GEMM_ACT_PAIR | _PAIR_FLAGS[act], splits, fused)


def act_mul(x, act="silu", out=None):
    """act(x[:, :I]) * x[:, I:2I]; `out` may be a column range of a wider matrix."""
    if not x.is_cuda:
        y = ref.act_mul(x, act)
        return y if out is None else out.copy_(y)
    T, two_i = x.shape
    if out is not None or x.dtype != torch.bfloat16 or act not in ("silu", "gelu", "gelu_tanh"):
        if out is None:
            out = torch.empty(T, two_i // 2, dtype=x.dtype, device=x.device)
        assert x.stride(1) == 1 and out.stride(1) == 1 and out.dtype == x.dtype
        _lib.check(_lib.lib().ogb_act_mul_rows(_ptr(x), x.stride(0), _ptr(out), out.stride(0), T, two_i // 2, _ACT[act], int(x.dtype == torch.float32),
                                              _stream()), "act_mul_rows")
        return out
    out = torch.empty(T, two_i // 2, dtype=x.dtype, device=x.device)
    _lib.check(_lib.lib().ogb_act_mul(_ptr(x), _ptr(out), T, two_i // 2, _ACT[act], _stream()), "act_mul")
    return out


def short_conv(bcx, weight, bias, cache, slots, positions, cu_seqlens, past_lens, block_table, block_size: int):
    """Gated short depthwise convolution of a hybrid (LFM2) layer over packed sequences; appends b * x of this step's tokens
    to the paged `cache` [slots, C] (see ops/reference.py::short_conv for the definition).  Returns [T, C]."""
    if not bcx.is_cuda:
        return ref.short_conv(bcx, weight, bias, cache, slots, positions, cu_seqlens, past_lens, block_table, block_size)
    T, C = bcx.shape[0], weight.shape[0]
    assert bcx.dtype == torch.bfloat16 and bcx.stride(1) == 1 and weight.is_contiguous() and cache.is_contiguous()
    assert block_table.stride(1) == 1
    out = torch.empty(T, C, dtype=bcx.dtype, device=bcx.device)
    _lib.check(_lib.lib().ogb_short_conv(_ptr(bcx), bcx.stride(0), _ptr(weight), _ptr(bias), _ptr(cache), _ptr(slots), _ptr(positions),
                                        _ptr(cu_seqlens), _ptr(past_lens), _ptr(block_table), block_table.stride(0), int(block_size),
                                        _ptr(out), T, past_lens.shape[0], C, weight.shape[1], _stream()), "short_conv")
    return out


def causal_conv(x, weight, bias, cache, slots, positions, cu_seqlens, past_lens, block_table, block_size: int, silu: bool = True):
    """Causal depthwise convolution (no gates) of the recurrent layer kinds over packed sequences, with the window of earlier
    positions read from the paged `cache` [slots, C] that this step's rows are appended to; optional SiLU.  x [T, C] may be a
    column slice of a wider tensor, `cache` a column range of wider rows.  Returns [T, C] in x's dtype."""
    if not x.is_cuda:
        ones = torch.ones_like(x)
        y = short_conv(torch.cat([ones, ones, x], dim=1).contiguous(), weight, bias, cache, slots, positions, cu_seqlens, past_lens, block_table, block_size)
        return torch.nn.functional.silu(y.float()).to(x.dtype) if silu else y
    T, C = x.shape[0], weight.shape[0]
    assert weight.is_contiguous() and cache.stride(1) == 1 and block_table.stride(1) == 1 and x.stride(1) == 1
    assert weight.dtype == x.dtype and cache.dtype == x.dtype
    out = torch.empty(T, C, dtype=x.dtype, device=x.device)
    args = (_ptr(slots), _ptr(positions), _ptr(cu_seqlens), _ptr(past_lens), _ptr(block_table), block_table.stride(0), int(block_size), _ptr(out), T,
            past_lens.shape[0], C, weight.shape[1])
    if x.dtype == torch.float32 or C % 8 or x.stride(0) % 8 or cache.stride(0) % 8 or (x.data_ptr() | cache.data_ptr()) % 16 or weight.shape[1] > 16:
        _lib.check(_lib.lib().ogb_causal_conv_rows(_ptr(x), x.stride(0), _ptr(weight), _ptr(bias), _ptr(cache), cache.stride(0), *args, int(silu),
                                                  int(x.dtype == torch.float32), _stream()), "causal_conv_rows")
        return out
    _lib.check(_lib.lib().ogb_causal_conv(_ptr(x), x.stride(0), _ptr(weight), _ptr(bias), _ptr(cache), *args, cache.stride(0), int(silu), _stream()),
               "causal_conv")
    return out


def gated_delta(q, k, v, g, beta, state, slots, cu_seqlens, past_lens, max_q_len: int = 0):
    """Gated-delta-rule recurrence of a linear-attention layer over packed sequences (see ops/reference.py::gated_delta).
    state [slots, Hv, dk, dv] fp32 is updated in place.  max_q_len: most tokens of one request (1 selects the decode kernel, 0: not
    known)."""
    if not q.is_cuda:
        return ref.gated_delta(q, k, v, g, beta, state, slots, cu_seqlens, past_lens)
    T, Hk, dk = q.shape
    Hv, dv = v.shape[1], v.shape[2]
    assert q.dtype == torch.bfloat16 and k.dtype == torch.bfloat16 and v.dtype == torch.bfloat16 and state.dtype == torch.float32
    assert q.is_contiguous() and k.is_contiguous() and v.is_contiguous() and state.is_contiguous()
    gf, bf = g.float().contiguous(), beta.float().contiguous()
    out = torch.empty(T, Hv, dv, dtype=torch.bfloat16, device=q.device)
    B = past_lens.shape[0]
    _lib.check(_lib.lib().ogb_gated_delta(_ptr(q), _ptr(k), _ptr(v), _ptr(gf), _ptr(bf), _ptr(state), _ptr(slots), _ptr(cu_seqlens), _ptr(past_lens),
                                          _ptr(out), B, Hk, Hv, dk, dv, int(max_q_len), _stream()), "gated_delta")
    return out


def gated_delta_layer(conv, proj, cd, vd, Hk, Hv, dk, dv, neg_exp_a, dt_bias, norm_w, norm_eps, state, slots, cu_seqlens, past_lens,
                      max_q_len: int = 0, l2_eps: float = 0.0, out=None):
    """The part of a gated-delta-net layer between its convolution and its output projection, as two kernels on CUDA tensors (bf16 or
    fp32): conv [T, cd] = silu(conv1d([q | k | v])), proj [T, cd + vd + 2 Hv] = the input projection [qkv | z | b | a].  q and k are
    L2-normalised per head (q also scaled by dk^-0.5), beta = sigmoid(b), log-decay = neg_exp_a * softplus(a + dt_bias), the
    recurrence updates `state` in place, and the result is RMS-normalised per value head, weighted and gated by silu(z).
    l2_eps > 0: unit vectors are x / sqrt(sum(x^2) + l2_eps), else x / max(|x|, 1e-6).  state [slots, Hv * dk * dv (or more)]: a slot's
    state is dense, slots may be further apart.  Returns [T, Hv * dv] (`out`: a matrix, or a column range, to write it to)."""
    T = conv.shape[0]
    assert conv.is_cuda and conv.dtype == proj.dtype and conv.dtype in (torch.bfloat16, torch.float32) and conv.stride(1) == 1 and proj.stride(1) == 1
    assert state.dtype == torch.float32 and state[0].numel() >= Hv * dk * dv and state[0].is_contiguous()
    kd, f32 = Hk * dk, int(conv.dtype == torch.float32)
    o = torch.empty(T, Hv, dv, dtype=conv.dtype, device=conv.device)
    B = past_lens.shape[0]
    _lib.check(_lib.lib().ogb_gated_delta_fused(_ptr(conv), conv.stride(0), 0, kd, 2 * kd, _ptr(proj), proj.stride(0), cd + vd, cd + vd + Hv,
                                                _ptr(neg_exp_a), _ptr(dt_bias), float(dk) ** -0.5, float(l2_eps), _ptr(state), state.stride(0),
                                                _ptr(slots), _ptr(cu_seqlens), _ptr(past_lens), _ptr(o), B, Hk, Hv, dk, dv, int(max_q_len), f32,
                                                _stream()), "gated_delta_fused")
    if out is None:
        out = torch.empty(T, Hv * dv, dtype=conv.dtype, device=conv.device)
    z = proj[:, cd:cd + vd]
    _lib.check(_lib.lib().ogb_gdn_gate_norm(_ptr(o), _ptr(z), proj.stride(0), _ptr(norm_w), float(norm_eps), _ptr(out), out.stride(0), T, Hv, dv, f32,
                                            _stream()), "gdn_gate_norm")
    return out


def mamba2_layer(conv, proj, heads, groups, P, N, dt_bias, neg_a, Dv, norm_w, norm_eps, state, slots, cu_seqlens, past_lens):
    """The part of a Mamba-2 layer between its convolution and its output projection, as two kernels on bf16 CUDA tensors:
    conv [T, I + 2 G N] = silu(conv1d([x | B | C])), proj [T, I + conv width + heads] = the input projection [z | xBC | dt].
    step = softplus(dt + dt_bias), the scan updates `state` in place, y * silu(z) is RMS-normalised over the whole width I = heads * P
    and weighted.  Returns [T, I]."""
    T = conv.shape[0]
    I = heads * P
    assert conv.is_cuda and conv.dtype == torch.bfloat16 and proj.dtype == torch.bfloat16 and conv.stride(1) == 1 and proj.stride(1) == 1
    y = torch.empty(T, I, dtype=torch.bfloat16, device=conv.device)
    dt_raw = proj[:, I + conv.shape[1]:]
    _lib.check(_lib.lib().ogb_mamba2_scan_fused(_ptr(conv), conv.stride(0), _ptr(dt_raw), proj.stride(0), _ptr(dt_bias), _ptr(neg_a), _ptr(Dv),
                                                _ptr(state), _ptr(slots), _ptr(cu_seqlens), _ptr(past_lens), _ptr(y), past_lens.shape[0], heads,
                                                groups, P, N, _stream()), "mamba2_scan_fused")
    out = torch.empty(T, I, dtype=torch.bfloat16, device=conv.device)
    _lib.check(_lib.lib().ogb_mamba_gate_norm(_ptr(y), _ptr(proj), proj.stride(0), _ptr(norm_w), float(norm_eps), _ptr(out), T, I, _stream()),
               "mamba_gate_norm")
    return out


def mamba2_scan(x, dt, neg_a, Bm, Cm, Dv, state, slots, cu_seqlens, past_lens):
    """Mamba-2 selective scan of a state-space layer over packed sequences (see ops/reference.py::mamba2_scan).
    state [slots, heads, N, P] fp32 is updated in place."""
    if not x.is_cuda:
        return ref.mamba2_scan(x, dt, neg_a, Bm, Cm, Dv, state, slots, cu_seqlens, past_lens)
    T, heads, P = x.shape
    groups, N = Bm.shape[1], Bm.shape[2]
    assert x.dtype == torch.bfloat16 and Bm.dtype == torch.bfloat16 and Cm.dtype == torch.bfloat16 and state.dtype == torch.float32
    assert x.is_contiguous() and Bm.is_contiguous() and Cm.is_contiguous() and state.is_contiguous()
    dtf, af, df = dt.float().contiguous(), neg_a.float().contiguous(), Dv.float().contiguous()
    out = torch.empty(T, heads, P, dtype=torch.bfloat16, device=x.device)
    _lib.check(_lib.lib().ogb_mamba2_scan(_ptr(x), _ptr(dtf), _ptr(af), _ptr(Bm), _ptr(Cm), _ptr(df), _ptr(state), _ptr(slots), _ptr(cu_seqlens),
                                          _ptr(past_lens), _ptr(out), past_lens.shape[0], heads, groups, P, N, _stream()), "mamba2_scan")
    return out


def copy_state_slots(src: torch.Tensor, dst: torch.Tensor, src_slots, dst_slots) -> None:
    """dst[:, dst_slots[i]] = src[:, src_slots[i]] for recurrent-state pools [layers, slots, ...] fp32 of the same shape (snapshots
    of linear-attention states around a speculative round)."""
    assert src.shape == dst.shape and src.dtype == dst.dtype == torch.float32 and src.is_contiguous() and dst.is_contiguous()
    ss = torch.as_tensor(src_slots, dtype=torch.int32, device=src.device).reshape(-1)
    ds = torch.as_tensor(dst_slots, dtype=torch.int32, device=src.device).reshape(-1)
    assert ss.numel() == ds.numel()
    if ss.numel() == 0:
        return
    if not src.is_cuda:
        dst[:, ds.long()] = src[:, ss.long()]
        return
    L, S = src.shape[0], src.shape[1]
    elems = src[0, 0].numel()
    _lib.check(_lib.lib().ogb_copy_state_slots(_ptr(src), _ptr(dst), L, S, elems, _ptr(ss), _ptr(ds), ss.numel(), _stream()), "copy_state_slots")


def decode_advance(sampled, input_ids, positions, past_lens, slot_mapping, sample_pos, block_table, block_size: int):
    """In place: the packed inputs of a one-token-per-request step become those of the next step (see
    csrc/elementwise.cu::decode_advance_kernel).  block_table [B, cols] int32, everything else [B] int32."""
    B = sampled.shape[0]
    if DEBUG_BOUNDS:
        _check_index("decode_advance", "positions + 1 (block-table column)", positions[:B] + 1, block_table.shape[1] * block_size)
    if not sampled.is_cuda:
        pos = positions[:B] + 1
        input_ids[:B] = sampled
        positions[:B] = pos
        past_lens[:B] += 1
        sample_pos[:B] += 1
        col = (pos // block_size).long()
        blk = torch.where(col < block_table.shape[1], block_table[torch.arange(B), col.clamp(max=block_table.shape[1] - 1)], torch.full_like(pos, -1))
        slot_mapping[:B] = torch.where(blk < 0, torch.full_like(pos, -1), blk * block_size + pos % block_size)
        return
    assert block_table.stride(1) == 1
    _lib.check(_lib.lib().ogb_decode_advance(_ptr(sampled), _ptr(input_ids), _ptr(positions), _ptr(past_lens), _ptr(slot_mapping),
                                            _ptr(sample_pos), _ptr(block_table), block_table.stride(0), int(block_size), B, _stream()),
               "decode_advance")


def activation(x, act="gelu"):
    """Elementwise activation of a bf16 tensor (the fc1 -> act -> fc2 MLPs of phi and gpt2)."""
    if not x.is_cuda:
        return ref.activation(x, act)
    x = x.contiguous()
    out = torch.empty_like(x)
    _lib.check(_lib.lib().ogb_act(_ptr(x), _ptr(out), x.numel(), _ACT[act], _stream()), "activation")
    return out


# ------------------------------------------------------------------------------------------ mixture of experts
def interleave_experts_gate_up(w: torch.Tensor, fused_interleaved: bool = True, block: int = 64) -> torch.Tensor:
    """Per-expert gate/up rows ([E, 2I, ...]; fused_interleaved: even rows = gate, odd rows = up, else [gate; up])
    -> per expert blocks of 64 gate rows followed by the 64 up rows of the same features."""
    E, two_i = w.shape[0], w.shape[1]
    inter = two_i // 2
    assert inter % block == 0
    if fused_interleaved:
        g, u = w[:, 0::2], w[:, 1::2]
    else:
        g, u = w[:, :inter], w[:, inter:]
    g = g.reshape(E, inter // block, 1, block, *w.shape[2:])
    u = u.reshape(E, inter // block, 1, block, *w.shape[2:])
    return torch.cat([g, u], dim=2).reshape(w.shape).contiguous()


class MoePlan:
    """Device-side routing of one MoE layer call (no host readback): which expert serves which sorted row."""
    __slots__ = ("T", "k", "E", "bt", "max_tiles", "topk_idx", "topk_w", "expert_offsets", "sorted_token", "inv_pos", "tile_expert",
                 "tile_row0", "tile_rows", "num_tiles")


def moe_route(router_logits: torch.Tensor, k: int, mode: int = 0, expert_range=None, token_tile: int = 0, topk=None, shared: bool = False, correction=None,
              groups: int = 1, keep: int = 1, scale: float = 1.0) -> MoePlan:
    """router_logits [T, E] fp32 -> MoePlan (top-k, routing weights, rows grouped by expert, GEMM tile list).
    mode 0: softmax over the selected logits; 1: softmax over all experts; 2: the latter renormalised; 3: the selected sigmoid scores divided by their
    sum, times `scale`, the selection by score + correction (fp32 [E]) within the `keep` best of `groups` groups.
    expert_range (lo, hi): only these experts are local (expert parallelism).  topk = (idx int32 [T, k], weights fp32 [T, k]):
    a selection made elsewhere (PhiMoE's sparse mixer); only the grouping by expert is computed.  shared: every token is also served by
    expert E, with weight 1 (the plan then has E + 1 experts and k + 1 of them per token)."""
    assert router_logits.is_cuda and router_logits.dtype == torch.float32 and router_logits.stride(-1) == 1
    T, routed = router_logits.shape
    top, k, E = k, k + int(shared), routed + int(shared)
    L = _lib.lib()
    dev = router_logits.device
    lo, hi = expert_range if expert_range is not None else (0, E)
    assert not shared or (topk is None and (lo, hi) == (0, E))
    pl = MoePlan()
    n = T * k
    bt = token_tile or L.ogb_gemm_token_tile(max(1, min(T, -(-2 * n // max(1, hi - lo)))), 0)
    pl.T, pl.k, pl.E, pl.bt = T, k, E, bt
    pl.max_tiles = L.ogb_moe_max_tiles(n, hi - lo, bt)
    i32 = dict(dtype=torch.int32, device=dev)
    if topk is not None:
        pl.topk_idx, pl.topk_w = topk
        assert pl.topk_idx.dtype == torch.int32 and pl.topk_w.dtype == torch.float32 and pl.topk_idx.shape == (T, k)
    else:
        pl.topk_idx = torch.empty(T, k, **i32)
        pl.topk_w = torch.empty(T, k, dtype=torch.float32, device=dev)
    pl.expert_offsets = torch.empty(E + 1, **i32)
    pl.sorted_token = torch.empty(n, **i32)
    pl.inv_pos = torch.empty(T, k, **i32)
    tiles = torch.empty(3 * pl.max_tiles + 1, **i32)
    pl.tile_expert, pl.tile_row0, pl.tile_rows = tiles[:pl.max_tiles], tiles[pl.max_tiles:2 * pl.max_tiles], tiles[2 * pl.max_tiles:3 * pl.max_tiles]
    pl.num_tiles = tiles[3 * pl.max_tiles:]
    if mode == 3:
        assert topk is None and not shared and correction.dtype == torch.float32 and correction.numel() == E
        _lib.check(L.ogb_moe_topk_grouped(_ptr(router_logits), router_logits.stride(0), T, E, k, _ptr(correction), int(groups), int(keep), float(scale),
                                          _ptr(pl.topk_idx), _ptr(pl.topk_w), _stream()), "moe_topk_grouped")
    elif topk is None:
        _lib.check(L.ogb_moe_topk(_ptr(router_logits), router_logits.stride(0), T, routed, top, mode, int(shared), _ptr(pl.topk_idx), _ptr(pl.topk_w), _stream()),
                   "moe_topk")
    _lib.check(L.ogb_moe_sort(_ptr(pl.topk_idx), T, k, E, lo, hi, bt, _ptr(pl.expert_offsets), _ptr(pl.sorted_token), _ptr(pl.inv_pos),
                              _ptr(pl.tile_expert), _ptr(pl.tile_row0), _ptr(pl.tile_rows), _ptr(pl.num_tiles), pl.max_tiles, _stream()),
               "moe_sort")
    return pl


def moe_fp4_reads_rows(w, plan: MoePlan) -> bool:
    """True when moe_gemm over these packed experts takes the un-gathered bf16 rows plus the plan's row map (row_map=True)."""
    return isinstance(w, Fp4Experts) and w.half and bool(_lib.lib().ogb_moe_fp4_reads_row_map(plan.bt, w.K, 1))


MOE_ACTS = {"relu2": 1 + _ACT["relu2"]}      # activations of experts without a gate matrix (act_kind of moe_gemm with pair=False)


def moe_gemm(xs: torch.Tensor, w: torch.Tensor, plan: MoePlan, bias=None, act_kind: int = 0, alpha: float = 1.0, limit: float = 0.0,
             out_dtype=torch.bfloat16, row_map: bool = False, pair: bool = True):
    """Grouped expert GEMM over rows sorted by expert.  xs [T*k, K] bf16; w [E, N, K] bf16; bias [E, N].
    act_kind 0: plain; 1: silu(gate)*up; 2: clamped SwiGLU(alpha, limit) — both need the 64-row gate/up blocks
    of interleave_experts_gate_up and return N/2 columns.  pair=False: act_kind is 0 or an entry of MOE_ACTS, for every column."""
    E, N, K = w.shape
    assert xs.is_cuda and xs.stride(-1) == 1
    ws = workspace(xs.device)
    if isinstance(w, Fp4Experts):
        # MXFP4 experts stay packed in HBM; the kernel expands each tile in shared memory (csrc/gemm_fp4.cu).  The fp16 form
        # takes fp16 rows (ops.gather_rows(..., f16=True) or the previous grouped GEMM with out_dtype=torch.float16).
        # row_map: xs holds the bf16 token rows [T, K] as they are; the kernel reads sorted row r from xs[plan.sorted_token[r]]
        assert out_dtype in (torch.bfloat16, torch.float16)
        assert xs.dtype == (torch.bfloat16 if row_map else (torch.float16 if w.half else torch.bfloat16))
        rows = plan.T * plan.k if row_map else xs.shape[0]
        out = torch.empty(rows, N // 2 if act_kind else N, dtype=out_dtype, device=xs.device)
        flags = (GEMM_ACT_PAIR if act_kind else 0) | (16 if w.half else 0) | (32 if out_dtype == torch.float16 else 0)
        rc = _lib.lib().ogb_moe_gemm_fp4(_ptr(xs), xs.stride(0), _ptr(w.packed), _ptr(out), out.stride(0), rows, N, K, E, _ptr(bias),
                                         flags, int(act_kind), float(alpha), float(limit),
                                         _ptr(plan.tile_expert), _ptr(plan.tile_row0), _ptr(plan.tile_rows), _ptr(plan.num_tiles),
                                         plan.max_tiles, plan.bt, plan.T, _ptr(plan.sorted_token) if row_map else None, ws.status,
                                         _stream())   # plan.T: an expert sees a token at most once
        _lib.check(rc, "moe_gemm_fp4")
        return out
    assert xs.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.is_contiguous()
    pair = pair and act_kind != 0
    out = torch.empty(xs.shape[0], N // 2 if pair else N, dtype=torch.bfloat16, device=xs.device)
    rc = _lib.lib().ogb_moe_gemm(_ptr(xs), xs.stride(0), _ptr(w), K, _ptr(out), out.stride(0), xs.shape[0], N, K, E, _ptr(bias),
                                 GEMM_ACT_PAIR if pair else 0, int(act_kind), float(alpha), float(limit), _ptr(plan.tile_expert),
                                 _ptr(plan.tile_row0), _ptr(plan.tile_rows), _ptr(plan.num_tiles), plan.max_tiles, plan.bt, ws.status,
                                 _stream())
    _lib.check(rc, "moe_gemm")
    return out


def moe_gemm_simt(xs: torch.Tensor, w: torch.Tensor, plan: MoePlan, mapped: bool = False) -> torch.Tensor:
    """Grouped expert product in plain arithmetic (fp32, or bf16 sizes TMA cannot address): w [E, N, K]; xs holds the rows sorted by expert,
    or (mapped) the token rows, read through the plan.  Returns [T * k, N] in xs's type."""
    E, N, K = w.shape
    assert xs.is_cuda and xs.dtype == w.dtype and xs.stride(1) == 1 and w.is_contiguous() and xs.dtype in (torch.float32, torch.bfloat16)
    assert plan.bt <= 64 and xs.shape[1] == K
    out = torch.empty(plan.T * plan.k, N, dtype=xs.dtype, device=xs.device)
    _lib.check(_lib.lib().ogb_moe_gemm_simt(_ptr(xs), xs.stride(0), _ptr(w), _ptr(out), N, N, K, _ptr(plan.tile_expert), _ptr(plan.tile_row0),
                                           _ptr(plan.tile_rows), _ptr(plan.num_tiles), plan.max_tiles, plan.bt, _ptr(plan.sorted_token) if mapped else None,
                                           int(xs.dtype == torch.float32), _stream()), "moe_gemm_simt")
    return out


def expert_act(gu: torch.Tensor, kind: str, alpha: float = 1.702, limit: float = 0.0) -> torch.Tensor:
    """Activation of expert rows whose columns alternate (gate, up): [n, 2 I] -> [n, I]; of rows without gates ("relu2"): [n, I] -> [n, I]."""
    assert gu.is_cuda and gu.is_contiguous()
    n, inter = gu.shape[0], gu.shape[1] // (1 if kind == "relu2" else 2)
    out = torch.empty(n, inter, dtype=gu.dtype, device=gu.device)
    _lib.check(_lib.lib().ogb_expert_act(_ptr(gu), _ptr(out), n, inter, {"silu": 0, "clamped": 1, "relu2": 2}[kind], float(alpha), float(limit),
                                        int(gu.dtype == torch.float32), _stream()), "expert_act")
    return out


def moe_combine(y: torch.Tensor, plan: MoePlan, residual=None) -> torch.Tensor:
    """out[t] = (residual[t]) + sum_j w[t, j] * y[row(t, j)]; rows of experts that are not local are skipped."""
    out = torch.empty(plan.T, y.shape[1], dtype=torch.bfloat16, device=y.device)
    rc = _lib.lib().ogb_moe_combine(_ptr(y), y.stride(0), _ptr(plan.inv_pos), _ptr(plan.topk_w), plan.T, plan.k, y.shape[1], _ptr(residual),
                                    residual.stride(0) if residual is not None else 0, _ptr(out), out.stride(0), _stream())
    _lib.check(rc, "moe_combine")
    return out


# ------------------------------------------------------------------------------------------ RoPE + KV append
def rope_kv_append(qkv, positions, slots, cos_cache, sin_cache, k_cache, v_cache, Hq, Hkv, D, rot, interleaved=False,
                   q_norm_w=None, k_norm_w=None, norm_eps=1e-6, positions3=None, mrope_section=None, mrope_interleaved=False):
    """positions3 [3, T] int32 + mrope_section (rotary pairs per component: temporal, height, width): multimodal RoPE, the
    pairs of each section rotate by their own position component.  mrope_interleaved: the components alternate pair by pair
    (t h w t h w ... while a component has pairs left) instead of occupying three contiguous ranges."""
    _check_index("rope_kv_append", "slots", None if slots is None else slots[:qkv.shape[0]], k_cache.shape[0] if k_cache is not None else 0, -1)
    if cos_cache is not None:
        _check_index("rope_kv_append", "positions", positions[:qkv.shape[0]] if positions3 is None else positions3, cos_cache.shape[0])
    if not qkv.is_cuda:
        return ref.rope_kv_append(qkv, positions, slots, cos_cache, sin_cache, k_cache, v_cache, Hq, Hkv, D, rot, interleaved,
                                  q_norm_w, k_norm_w, norm_eps, positions3, mrope_section, mrope_interleaved)
    assert qkv.dtype == torch.bfloat16 and qkv.stride(1) == 1
    assert cos_cache is None or cos_cache.dtype == torch.float32
    T = qkv.shape[0]
    max_pos = cos_cache.shape[0] if cos_cache is not None else 1
    kv_bits = 8 if k_cache.dtype == torch.int8 else 16      # an int8 cache has rows of D values + inline scale (D + 16 bytes)
    rc = _lib.lib().ogb_rope_kv_append_bits(_ptr(qkv), qkv.stride(0), _ptr(positions), _ptr(slots), _ptr(cos_cache), _ptr(sin_cache),
                                            _ptr(k_cache), _ptr(v_cache), _ptr(q_norm_w), _ptr(k_norm_w), float(norm_eps), T, Hq, Hkv,
                                            D, int(rot if cos_cache is not None else 0), int(interleaved), max_pos, kv_bits,
                                            _ptr(positions3.contiguous()) if positions3 is not None else None,
                                            (0 if positions3 is None else -3 * int(mrope_section[1]) if mrope_interleaved else int(mrope_section[0])),
                                            (0 if positions3 is None else 3 * int(mrope_section[2]) if mrope_interleaved
                                             else int(mrope_section[0] + mrope_section[1])), _stream())
    _lib.check(rc, "rope_kv_append")
    return qkv


def qkv_prep(proj, Hq, Hkv, dim, key_row, value_row, q_norm_w, k_norm_w, eps, positions, cos, sin, slots, k_cache, v_cache, Hv=None, talk=None,
             mixed=None):
    """Between the projection [Hq queries | Hkv keys | Hv (None: Hkv) values | ...] of an attention layer and its attention: RMS norm of every query and
    key head over its `dim` columns (weights fp32 [dim] or None), rotation of the first 2 * cos.shape[1] of them (cos / sin fp32 [positions,
    rot / 2], or None), queries in place, keys and values to row slots[t] of the caches [slots, Hkv, key_row] and [slots, Hv, value_row]
    (slot < 0: to no row).  Any sizes, bf16 or fp32.  talk [Hq, Hq] fp32: the queries stay; row t of `mixed` [T, Hq * Hkv * key_row] gets, for head h and
    key head c, the sum of talk[h, g] times query g over the heads g of c's group."""
    Hv = Hv or Hkv
    _check_index("qkv_prep", "slots", slots[:proj.shape[0]], k_cache.shape[0], -1)
    if cos is not None:
        _check_index("qkv_prep", "positions", positions[:proj.shape[0]], cos.shape[0])
    if not proj.is_cuda:
        return ref.qkv_prep(proj, Hq, Hkv, dim, key_row, value_row, q_norm_w, k_norm_w, eps, positions, cos, sin, slots, k_cache, v_cache, Hv, talk, mixed)
    assert talk is None or (talk.dtype == torch.float32 and talk.is_contiguous() and mixed.is_contiguous() and mixed.dtype == proj.dtype and
                            mixed.shape == (proj.shape[0], Hq * Hkv * key_row))
    assert proj.stride(1) == 1 and k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.dtype == v_cache.dtype == proj.dtype
    assert proj.dtype in (torch.bfloat16, torch.float32) and all(w is None or w.dtype == torch.float32 for w in (q_norm_w, k_norm_w, cos, sin))
    _lib.check(_lib.lib().ogb_qkv_prep(_ptr(proj), proj.stride(0), Hq, Hkv, Hv, dim, key_row, value_row, _ptr(q_norm_w), _ptr(k_norm_w), float(eps),
                                      _ptr(positions), _ptr(cos), _ptr(sin), 2 * cos.shape[1] if cos is not None else 0,
                                      cos.shape[0] if cos is not None else 1, _ptr(slots), _ptr(k_cache), _ptr(v_cache), proj.shape[0], _ptr(talk), _ptr(mixed),
                                      int(proj.dtype == torch.float32), _stream()), "qkv_prep")
    return proj


# ------------------------------------------------------------------------------------------ attention
def choose_kv_splits(batch: int, Hkv: int, max_q_len: int, max_kv_len: int, sm_count: int = 148, group: int = 1, ordered: bool = False):
    """(splits, kv_chunk) of a paged-attention launch.  A launch whose (request, kv head) grid already fills the GPU
    twice over is not split (measured on B200: at 64 requests x 8 heads any split costs more in partial traffic and
    the merge than it gains in balance).  Smaller decode-sized launches split every request's keys into fixed chunks
    of 64..512 keys sized for about four CTAs per SM; other launches: (1, 0).

    ordered: the caller issues the requests longest first.  Then every request is divided evenly into as many parts as
    bring the launch to about 1.75 waves of CTAs - measured on B200 with 64 requests of 192..2112 keys and 4 / 2 / 1 kv
    heads per GPU (the tensor-parallel shapes): 2 parts 35.3 us against 43.1 us for fixed chunks, 4 parts 25.1 against
    29.4, 4 parts 18.7 against 22.0."""
    ctas = max(1, batch * Hkv)
    if ordered and ctas >= 32 and max_q_len * group <= 16 and max_kv_len > 128:
        s = int(round(1.75 * 2 * sm_count / ctas))
        s = max(1, min(4, s, max_kv_len // 256))     # more than 4 parts: the pieces get too short (1 kv head: 8 parts 20.5 us, 16 parts 27.7)
        return s, 0
    if max_q_len * group > 16 or max_kv_len <= 128 or ctas >= 2 * sm_count:
        return 1, 0
    chunks_wanted = max(1, (4 * sm_count + ctas - 1) // ctas)
    chunk = (max_kv_len + chunks_wanted - 1) // chunks_wanted
    chunk = min(512, max(64, (chunk + 63) // 64 * 64))
    splits = min(64, (max_kv_len + chunk - 1) // chunk)
    if splits <= 1:
        return 1, 0
    chunk = ((max_kv_len + splits - 1) // splits + 63) // 64 * 64   # the splits must cover the bound
    return int(splits), int(chunk)


def choose_joint_splits(batch: int, Hq: int, max_q_len: int, span: int, cols: int) -> int:
    """Key splits of a launch for heads whose scores are mixed (one CTA per token and 32 heads; rows of `cols` columns).  Measured on B200 with requests of
    192..2112 keys, 4 key heads of 128: 1 request 16 splits 18.4 us, 16 requests 12 splits 26.1 us, 64 requests 6 splits 46.5 us (4: 50), 256 requests
    2 splits 116 us (1: 137).  8 key heads of 128 (one CTA per SM): 16 requests 12 splits 48 us, 64 requests 4 splits 102 us (6: 117), 256 in one 311 us
    (2: 335)."""
    ctas = max(1, batch * max_q_len * ((Hq + 31) // 32))
    return max(1, min(int(round((200 if ctas <= 32 else (400 if cols <= 512 else 256)) / ctas)), span // 32, 16))


TC_ATTENTION_MIN_ROWS = 128      # query rows (tokens x heads of a GQA group) from which a request takes the tcgen05 prefill kernel
_TC_ATTENTION = os.environ.get("OGB_ATTN_TC", "1") != "0"


def paged_attention(q, k_cache, v_cache, cu_seqlens, past_lens, block_table, block_size, Hq, Hkv, D, scale, window=0,
                    sinks=None, softcap=0.0, max_q_len=None, max_kv_len=None, splits=None, out=None, total_tokens=None, order=None,
                    min_q_len=None, vdim=None, chunk=0, gate=None, maps=1, diff=None, joint=False, out_scale=1.0):
    """q: [T, stride] with the Hq*D query columns first.  Returns [T, Hq*D].  total_tokens: the requests of this call only cover
    the first `total_tokens` rows of q (sizes the split-KV scratch).  min_q_len: shortest request of the call when the caller
    knows it (a call whose every request is long runs on the tensor-core prefill kernel alone).  vdim (layers with sizes of their own): width
    of a value head; chunk > 0: position p sees the keys from p // chunk * chunk on; gate [T, Hq]: each head's output is multiplied by its
    sigmoid, or [T, heads * vdim]: each output column.  maps = 2, diff = (lambda, post, eps, columns): differential attention - q holds Hq vectors of
    D / 2 columns, 2 h and 2 h + 1 for head h, a key head both maps' keys; returns the Hq / 2 heads (see csrc/kernels.h, ogb_attention_diff_merge),
    RMS-normed over the first `columns` of each.  joint: the key heads of a cache row are one key of D columns, which every query head (D wide) meets.
    The result is multiplied by out_scale."""
    _check_index("paged_attention", "block_table", block_table, k_cache.shape[0] // block_size, -1)
    _check_index("paged_attention", "cu_seqlens", cu_seqlens[:past_lens.shape[0] + 1], q.shape[0] + 1)
    if not q.is_cuda:
        o = ref.paged_attention(q, k_cache, v_cache, cu_seqlens, past_lens, block_table, block_size, Hq, Hkv, D, scale,
                                window, sinks, softcap, vdim, chunk, gate, maps, diff, joint, out_scale)
        return o if out is None else out.copy_(o)
    if vdim is not None or chunk > 0 or gate is not None or maps > 1 or joint or out_scale != 1.0:
        return _paged_attention_mixed(q, k_cache, v_cache, cu_seqlens, past_lens, block_table, block_size, Hq, Hkv, D, vdim or D, scale, window, chunk,
                                      sinks, softcap, gate, max_q_len, max_kv_len, splits, out, total_tokens, order, min_q_len, maps, diff, joint, out_scale)
    T = q.shape[0] if total_tokens is None else total_tokens
    B = past_lens.shape[0]
    if out is None:
        out = torch.empty(q.shape[0], Hq * D, dtype=q.dtype, device=q.device)
    if max_q_len is None:
        max_q_len = T
    G = Hq // Hkv
    ws = workspace(q.device)
    use_tc = (_TC_ATTENTION and max_q_len * G >= TC_ATTENTION_MIN_ROWS and k_cache.dtype == torch.bfloat16 and q.dtype == torch.bfloat16
              and out.stride(0) % 8 == 0 and _lib.lib().ogb_attention_tc_supported(D, block_size, 16, int(k_cache.shape[0])))
    if use_tc:
        all_long = min_q_len is not None and min_q_len * G >= TC_ATTENTION_MIN_ROWS
        if not all_long:
            # the short requests first (its split-KV combine pass may scribble on the rows of the long ones)
            paged_attention_small = _lib.lib().ogb_paged_attention_skip
            sp, ch = splits if isinstance(splits, tuple) else ((splits, 0) if splits else choose_kv_splits(
                B, Hkv, max_q_len, max_kv_len or 1024, group=G, ordered=order is not None))
            need = _lib.lib().ogb_attention_scratch_bytes(T, Hq, D, sp)
            scratch = ws.attn_scratch(need) if sp > 1 else None
            _lib.check(paged_attention_small(_ptr(q), q.stride(0), _ptr(k_cache), _ptr(v_cache), _ptr(cu_seqlens), _ptr(past_lens),
                                             _ptr(block_table), block_table.stride(0), block_size, _ptr(out), out.stride(0), _ptr(sinks),
                                             float(scale), float(softcap), int(window), B, T, int(max_q_len), Hq, Hkv, D, int(sp), int(ch),
                                             _ptr(scratch), scratch.numel() if scratch is not None else 0, int(k_cache.shape[0]),
                                             _ptr(order), ws.status, _stream(), TC_ATTENTION_MIN_ROWS), "paged_attention")
            if sp > 1:
                _lib.LAUNCH_COUNT += 1
        _lib.check(_lib.lib().ogb_attention_tc(_ptr(q), q.stride(0), _ptr(k_cache), _ptr(v_cache), _ptr(cu_seqlens), _ptr(past_lens),
                                               _ptr(block_table), block_table.stride(0), block_size, _ptr(out), out.stride(0), _ptr(sinks),
                                               float(scale), float(softcap), int(window), B, int(max_q_len), Hq, Hkv, D,
                                               TC_ATTENTION_MIN_ROWS, int(k_cache.shape[0]), ws.status, _stream()), "attention_tc")
        return out
    kv_chunk = 0
    if splits is None:
        splits, kv_chunk = choose_kv_splits(B, Hkv, max_q_len, max_kv_len or 1024, group=Hq // Hkv, ordered=order is not None)
    elif isinstance(splits, tuple):
        splits, kv_chunk = splits
    need = _lib.lib().ogb_attention_scratch_bytes(T, Hq, D, splits)
    scratch = ws.attn_scratch(need) if splits > 1 else None
    fn = _lib.lib().ogb_paged_attention_kv8 if k_cache.dtype == torch.int8 else _lib.lib().ogb_paged_attention
    rc = fn(_ptr(q), q.stride(0), _ptr(k_cache), _ptr(v_cache), _ptr(cu_seqlens), _ptr(past_lens),
                                        _ptr(block_table), block_table.stride(0), block_size, _ptr(out), out.stride(0),
                                        _ptr(sinks), float(scale), float(softcap), int(window), B, T, int(max_q_len),
                                        Hq, Hkv, D, int(splits), int(kv_chunk), _ptr(scratch),
                                        scratch.numel() if scratch is not None else 0, int(k_cache.shape[0]), _ptr(order), ws.status, _stream())
    _lib.check(rc, "paged_attention")
    if splits > 1:
        _lib.LAUNCH_COUNT += 1  # the combine kernel
    return out


def _paged_attention_mixed(q, k_cache, v_cache, cu_seqlens, past_lens, block_table, block_size, Hq, Hkv, dk, dv, scale, window, chunk, sinks, softcap,
                           gate, max_q_len, max_kv_len, splits, out, total_tokens, order, min_q_len, maps=1, diff=None, joint=False, out_scale=1.0):
    """paged_attention of layers with sizes of their own: the tensor-memory kernel for requests with at least TC_ATTENTION_MIN_ROWS query
    rows, the warp-MMA kernel for the others, plain arithmetic for fp32 and for sizes neither can address."""
    import ctypes
    T = q.shape[0] if total_tokens is None else total_tokens
    B = past_lens.shape[0]
    assert (maps == 1) == (diff is None) and maps <= 2 and (diff is None or sinks is None)
    if out is None:
        out = torch.empty(q.shape[0], Hq // maps * dv, dtype=q.dtype, device=q.device)
    max_q_len = max_q_len or T
    L, G, ws = _lib.lib(), Hq // Hkv, workspace(q.device)
    assert k_cache.is_contiguous() and v_cache.is_contiguous() and q.stride(1) == 1 and out.stride(1) == 1 and block_table.stride(1) == 1
    assert sinks is None or sinks.dtype == torch.float32
    assert gate is None or (gate.dtype == q.dtype and gate.stride(1) == 1 and gate.shape[1] in (Hq, Hq // maps * dv))
    wide = gate is not None and gate.shape[1] == Hq // maps * dv and (dv > 1 or maps > 1)
    in_kernel = gate if diff is None else None             # (a differential layer's gate belongs to the merge of its maps)
    layer = _lib.AttnLayer(Hq=Hq, Hkv=Hkv, dk=dk, dv=dv, window=int(window), chunk=int(chunk), gate_stride=gate.stride(0) if gate is not None else 0,
                           scale=float(scale), sinks=_ptr(sinks), gate=_ptr(in_kernel), gate_wide=int(wide), maps=maps, raw=int(diff is not None),
                           softcap=float(softcap or 0.0), joint=int(joint), out_scale=float(out_scale))

    def merge(part, sp, part_tokens):
        """Differential layers: the two maps' partial results of the call's tokens become the heads."""
        lam, post, eps, cols = diff
        _lib.check(L.ogb_attention_diff_merge(_ptr(part), int(sp), min(T, out.shape[0]), int(part_tokens), Hq // 2, dv, int(cols), float(lam), float(post),
                                              float(eps), _ptr(gate), gate.stride(0) if gate is not None else 0, _ptr(out), out.stride(0),
                                              int(out.dtype == torch.float32), _stream()), "attention_diff_merge")
        return out

    def part_bytes(tokens, sp):
        return int(sp) * tokens * Hq * (dv + 2) * 4
    inputs = (ctypes.byref(layer), _ptr(q), q.stride(0), _ptr(k_cache), _ptr(v_cache), _ptr(cu_seqlens), _ptr(past_lens), _ptr(block_table),
              block_table.stride(0), int(block_size), _ptr(out), out.stride(0), B)
    served = L.ogb_attention_joint_supported(dk, Hkv * dv) if joint else L.ogb_attention_mixed_supported(dk, dv)
    if (q.dtype == torch.float32 or not served or q.stride(0) % 8 or out.stride(0) % 2 or q.data_ptr() % 16 or out.data_ptr() % 4 or
            (joint and (dv % 8 or chunk > 0 or (wide and (gate.stride(0) % 2 or gate.data_ptr() % 4))))):
        # (the grid covers the rows of the whole matrix: rows of requests outside this call are skipped)
        n = q.shape[0]
        scratch = ws.attn_scratch(part_bytes(n, 1)) if diff is not None else None
        _lib.check(L.ogb_attention_simt(*inputs, n, _ptr(scratch), scratch.numel() if scratch is not None else 0, int(q.dtype == torch.float32), _stream()),
                   "attention_simt")
        return out if diff is None else merge(scratch, 1, n)
    slots = int(k_cache.shape[0])
    long_rows = TC_ATTENTION_MIN_ROWS
    use_tc = (_TC_ATTENTION and max_q_len * G >= long_rows and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0 and
              bool(L.ogb_attention_tc_joint_supported(dk, dv, int(block_size), slots) if joint else
                   L.ogb_attention_tc_mixed_supported(dk // maps, dv, int(block_size), slots)) and
              (not wide or diff is not None or (gate.stride(0) % 8 == 0 and gate.data_ptr() % 16 == 0)))
    sp, ch, scratch = 1, 0, None
    all_long = use_tc and min_q_len is not None and min_q_len * G >= long_rows
    if not all_long:
        # (first: with splits the combine pass leaves unspecified values in the rows of the long requests)
        if splits is None:
            span = max_kv_len or 1024
            if chunk > 0 or window > 0:
                span = min(span, (chunk or window) + 63)
            if joint:
                splits = choose_joint_splits(B, Hq, max_q_len, span, max(dk, Hkv * dv))
            else:
                splits = choose_kv_splits(B, Hkv, max_q_len, span, group=G, ordered=order is not None)
        sp, ch = splits if isinstance(splits, tuple) else (splits, 0)
    if sp > 1 or diff is not None:
        scratch = ws.attn_scratch(part_bytes(T, sp))
    if not all_long and joint:
        _lib.check(L.ogb_attention_joint(*inputs, T, int(max_q_len), int(sp), _ptr(scratch), scratch.numel() if scratch is not None else 0, _ptr(order),
                                         ws.status, _stream(), long_rows if use_tc else 0), "attention_joint")
        if sp > 1:
            _lib.LAUNCH_COUNT += 1      # the combine kernel
    elif not all_long:
        _lib.check(L.ogb_attention_mixed(*inputs, T, int(max_q_len), int(sp), int(ch), _ptr(scratch), scratch.numel() if scratch is not None else 0,
                                         _ptr(order), ws.status, _stream(), long_rows if use_tc else 0), "attention_mixed")
        if sp > 1 and diff is None:
            _lib.LAUNCH_COUNT += 1      # the combine kernel
    if use_tc:
        _lib.check(L.ogb_attention_tc_mixed(*inputs, int(max_q_len), long_rows, slots, int(sp), T, _ptr(scratch),
                                            scratch.numel() if scratch is not None else 0, ws.status, _stream()), "attention_tc_mixed")
    return out if diff is None else merge(scratch, sp, T)


# ------------------------------------------------------------------------------------------ recurrent mixers of declared stacks
MIN_GRU_STEP_TOKENS = 16    # portions of at most this many tokens are walked token by token


def min_gru(z, x, g, state, slots, cu_seqlens, past_lens, out, scale=1.0, max_q_len=0):
    """Gated average per column over packed sequences: S <- (1 - sigmoid(z)) S + sigmoid(z) * c(x) with c(x) = x + 1/2 for x >= 0 and sigmoid(x) below;
    out = S * silu(g) * scale.  z, x, g [T, W]: columns of one matrix; state [slots, W] fp32 (rows may be further apart), updated in place; a request whose
    past length is 0 starts from zero.  max_q_len: the most tokens a request feeds (0: unknown)."""
    if not z.is_cuda:
        return ref.min_gru(z, x, g, state, slots, cu_seqlens, past_lens, out, scale)
    T, W = z.shape
    assert z.dtype == x.dtype == g.dtype == out.dtype and z.stride() == x.stride() == g.stride() and z.stride(1) == out.stride(1) == 1
    assert state.dtype == torch.float32 and state.stride(1) == 1 and out.shape == (T, W)
    max_q_len = int(max_q_len or T)
    scratch = None
    if max_q_len > MIN_GRU_STEP_TOKENS:
        scratch = torch.empty(_lib.lib().ogb_min_gru_scratch_bytes(T, past_lens.shape[0], W), dtype=torch.uint8, device=z.device)
        _lib.LAUNCH_COUNT += 1
    _lib.check(_lib.lib().ogb_min_gru(_ptr(z), _ptr(x), _ptr(g), z.stride(0), _ptr(state), state.stride(0), _ptr(slots), _ptr(cu_seqlens), _ptr(past_lens),
                                     _ptr(out), out.stride(0), T, past_lens.shape[0], W, float(scale), max_q_len, _ptr(scratch),
                                     scratch.numel() if scratch is not None else 0, int(z.dtype == torch.float32), _stream()), "min_gru")
    return out


MLSTM_LONG_TOKENS = 24      # requests that feed at least this many tokens run in the chunk form of the matrix memories


def mlstm(proj, gates, gate_b, heads, dim, vdim, cap, norm_w, eps, state, slots, cu_seqlens, past_lens, out, max_q_len=0, min_q_len=0):
    """Matrix memories over packed sequences (see csrc/recurrent.cu): proj [T, queries | keys | values | output gate], gates fp32 [T, input | forget logits],
    their biases gate_b and the heads' norm weight fp32; state [slots, heads * (dim * vdim + dim + 1)] fp32, updated in place; out [T, heads * vdim].
    max_q_len, min_q_len: most and fewest tokens a request feeds (0: unknown)."""
    if not proj.is_cuda:
        return ref.mlstm(proj, gates, gate_b, heads, dim, vdim, cap, norm_w, eps, state, slots, cu_seqlens, past_lens, out)
    import ctypes
    nk, nv, es = heads * dim, heads * vdim, proj.element_size()
    assert proj.stride(1) == 1 and out.stride(1) == 1 and out.dtype == proj.dtype and gates.dtype == torch.float32 and gates.stride(1) == 1
    assert state.dtype == torch.float32 and state.stride(1) == 1 and state.shape[1] >= heads * (dim * vdim + dim + 1)
    at = proj.data_ptr()
    p = _lib.Mlstm(q=at, k=at + nk * es, v=at + 2 * nk * es, g=at + (2 * nk + nv) * es, gates=_ptr(gates), gate_b=_ptr(gate_b), norm_w=_ptr(norm_w),
                   out=_ptr(out), state=_ptr(state), slots=_ptr(slots), cu_seqlens=_ptr(cu_seqlens), past_lens=_ptr(past_lens), slot_stride=state.stride(0),
                   ld=proj.stride(0), ldg=gates.stride(0), ldo=out.stride(0), B=past_lens.shape[0], H=heads, d=dim, dv=vdim, T=proj.shape[0],
                   max_q_len=int(max_q_len or proj.shape[0]), fp32=int(proj.dtype == torch.float32), cap=float(cap), eps=float(eps))
    scratch = None
    if p.max_q_len >= MLSTM_LONG_TOKENS and not p.fp32 and p.ld % 8 == 0 and at % 16 == 0 and out.stride(0) % 2 == 0 and out.data_ptr() % 4 == 0:
        need = _lib.lib().ogb_mlstm_scratch_bytes(p.T, p.B, heads, dim, vdim)
        if need:
            scratch = torch.empty(need, dtype=torch.uint8, device=proj.device)
            p.scratch, p.scratch_bytes, p.long_tokens, p.all_long = _ptr(scratch), need, MLSTM_LONG_TOKENS, int(min_q_len >= MLSTM_LONG_TOKENS)
            _lib.LAUNCH_COUNT += 3 + (1 - p.all_long)
    _lib.check(_lib.lib().ogb_mlstm(ctypes.byref(p), _stream()), "mlstm")
    return out


# ------------------------------------------------------------------------------------------ latent attention
LATENT_LONG_TOKENS = 64      # requests that feed at least this many tokens attend on expanded keys and values (tensor-memory kernel)


def latent_shape(heads, dim, rot, vdim, kv_rank, rot_dims):
    return _lib.LatentShape(H=heads, dim=dim, rot=rot, vdim=vdim, R=kv_rank, rot_dims=rot_dims)


def _sh(shape):
    import ctypes
    return ctypes.byref(shape)


def latent_prep(proj, shape, norm_w, eps, positions, cos, sin, slots, cache):
    """`latent_prep_parts` of one projection [H heads of (dim | rot) | latent | shared rotary key].  In place: rotates the rotary part of every query head of proj ([H heads of (dim | rot)] then [latent | shared rotary key]), and
    writes the RMS-normalised latent and the rotated key of each token to its row of `cache` [slots, >= kv_rank + rot] (slot < 0: to no
    row).  cos / sin [positions, rot_dims / 2] fp32, or None for a layer that does not rotate."""
    _check_index("latent_prep", "slots", slots[:proj.shape[0]], cache.shape[0], -1)
    if cos is not None:
        _check_index("latent_prep", "positions", positions[:proj.shape[0]], cos.shape[0])
    n = shape.H * (shape.dim + shape.rot)
    latent_prep_parts(shape, eps, positions, cos, sin, q=proj[:, :n], down=proj[:, n:], norm_w=norm_w, slots=slots, cache=cache)
    return proj


def latent_prep_parts(shape, eps, positions, cos, sin, q=None, down=None, norm_w=None, slots=None, cache=None, cq=None, cq_w=None):
    """The steps around a latent-attention layer's projections, each where its matrix is given: q [T, H * (dim | rot)]: the rotary parts are rotated in
    place; down [T, latent | shared rotary key]: normed (weight norm_w) and rotated into `cache`; cq [T, q_rank]: RMS norm with weight cq_w in
    place (the queries' own latent)."""
    some = next(t for t in (q, down, cq) if t is not None)
    if not some.is_cuda:
        return ref.latent_prep_parts(shape, eps, positions, cos, sin, q, down, norm_w, slots, cache, cq, cq_w)
    assert all(t is None or (t.stride(1) == 1 and t.dtype == some.dtype) for t in (q, down, cq, cache))
    assert all(t is None or t.dtype == torch.float32 for t in (norm_w, cq_w)) and (down is None or (cache is not None and slots is not None))
    ld = lambda t: t.stride(0) if t is not None else 0
    _lib.check(_lib.lib().ogb_latent_prep(_ptr(q), ld(q), _ptr(down), ld(down), _ptr(cq), ld(cq), cq.shape[1] if cq is not None else 0, _ptr(cq_w),
                                         _sh(shape), _ptr(norm_w), float(eps), _ptr(positions), _ptr(cos), _ptr(sin),
                                         cos.shape[0] if cos is not None else 1, _ptr(slots), _ptr(cache), ld(cache), some.shape[0],
                                         int(some.dtype == torch.float32), _stream()), "latent_prep")


def gate_rows(x, gate):
    """x *= sigmoid(gate) in place; both [T, n] (column ranges of wider matrices)."""
    if not x.is_cuda:
        return x.copy_((x.float() * torch.sigmoid(gate.float())).to(x.dtype))
    assert x.stride(1) == 1 and gate.stride(1) == 1 and gate.shape == x.shape and gate.dtype == x.dtype
    _lib.check(_lib.lib().ogb_gate_rows(_ptr(x), x.stride(0), _ptr(gate), gate.stride(0), x.shape[0], x.shape[1], int(x.dtype == torch.float32), _stream()),
               "gate_rows")
    return x


def choose_latent_splits(batch: int, row_tiles: int, tile_rows: int, max_kv_len: int, window: int, sm_count: int = 148) -> int:
    """Key splits of a latent-attention launch: 3.5 CTAs per SM for 16-row tiles (two are resident at a time, the others even out requests of
    different lengths), 1.5 for taller tiles, each split at least two tiles of 32 keys.  Measured on B200 with requests of 192..2112 keys:
    16 heads, 64 requests 6 - 8 splits 36 us (4: 45), 256 requests 2 splits 96 us (1: 153, 3: 105); 32 heads, 64 requests longest first 4 splits
    55 us (3: 59, 6: 60), all of 2049 keys 95 us (3: 115, 6: 98)."""
    span = max_kv_len if window <= 0 else min(max_kv_len, window + 64)
    want = (3.5 if tile_rows <= 16 else 1.5) * sm_count / max(1, batch * row_tiles)
    return max(1, min(int(round(want)), span // 64, 32))


def latent_attention(qlat, proj, shape, cache, cu_seqlens, past_lens, block_table, block_size, scale, window=0, max_q_len=1, max_kv_len=1,
                     skip_q_len=0, splits=None, order=None, sinks=None):
    """Attention of every head over the shared latent rows: qlat [T, H * kv_rank] (queries with the key map folded in), the rotated
    query parts in proj.  window > 0: position p sees (p - window, p].  skip_q_len > 0: requests with at least that many tokens are
    not computed (their rows are unspecified).  order [B]: requests in the order in which their CTAs are issued.  sinks [H] fp32: a logit in each
    head's denominator.  Returns [T, H * kv_rank]."""
    _check_index("latent_attention", "block_table", block_table, cache.shape[0] // block_size, -1)
    if not qlat.is_cuda:
        return ref.latent_attention(qlat, proj, shape, cache, cu_seqlens, past_lens, block_table, block_size, scale, window, sinks)
    T, B, H, R = qlat.shape[0], past_lens.shape[0], shape.H, shape.R
    out = torch.empty_like(qlat)
    L = _lib.lib()
    f32 = qlat.dtype == torch.float32
    if (f32 or not L.ogb_latent_mma_supported(_sh(shape)) or proj.stride(0) % 8 or cache.stride(0) % 8 or
            (qlat.data_ptr() | proj.data_ptr() | cache.data_ptr()) % 16):
        _lib.check(L.ogb_latent_attention_simt(_ptr(qlat), _ptr(proj), proj.stride(0), _sh(shape), _ptr(cache), cache.stride(0), _ptr(cu_seqlens),
                                               _ptr(past_lens), _ptr(block_table), block_table.stride(0), int(block_size), _ptr(out), float(scale),
                                               int(window), _ptr(sinks), B, T, int(skip_q_len), int(f32), _stream()), "latent_attention_simt")
        return out
    q_len = min(max_q_len, skip_q_len - 1) if skip_q_len > 0 else max_q_len
    if splits is None:
        bm = L.ogb_latent_rows_per_tile(H, q_len)
        splits = choose_latent_splits(B, -(-H * q_len // bm), bm, max_kv_len, window)
    need = L.ogb_latent_scratch_bytes(T * H, R, splits)
    scratch = workspace(qlat.device).attn_scratch(need) if splits > 1 else None
    _lib.check(L.ogb_latent_attention(_ptr(qlat), _ptr(proj), proj.stride(0), _sh(shape), _ptr(cache), cache.stride(0), _ptr(cu_seqlens), _ptr(past_lens),
                                      _ptr(block_table), block_table.stride(0), int(block_size), _ptr(out), float(scale), int(window), _ptr(sinks), B, T,
                                      int(max_q_len), int(skip_q_len), int(splits), _ptr(scratch), scratch.numel() if scratch is not None else 0,
                                      _ptr(order), workspace(qlat.device).status, _stream()), "latent_attention")
    if splits > 1:
        _lib.LAUNCH_COUNT += 1      # the combine kernel
    return out


def latent_long_supported(shape, proj, cache, block_size: int) -> bool:
    return (proj.is_cuda and proj.dtype == torch.bfloat16 and bool(_lib.lib().ogb_attention_tc_latent_supported(shape.dim, shape.rot, shape.vdim)) and
            shape.R % 8 == 0 and proj.stride(0) % 8 == 0 and cache.stride(0) % 8 == 0)


class LatentPlan:
    """Where the long requests of a step put their expanded keys: per request a run of dense rows (a multiple of 16) for the cached
    positions its tokens can see."""
    __slots__ = ("rows", "row_base", "first_kv", "g_base", "g_first", "g_len", "g_req", "n_req", "max_q_len")

    def __init__(self, lens, window: int, device, min_tokens: int = LATENT_LONG_TOKENS):
        B = len(lens)
        base, first = np.full(B, -1, dtype=np.int32), np.zeros(B, dtype=np.int32)
        compact, rows, self.max_q_len = [], 0, 0
        for b, (past, n) in enumerate(lens):
            if n < min_tokens:
                continue
            lo = max(0, past - window + 1) // 16 * 16 if window > 0 else 0
            base[b], first[b] = rows, lo
            compact.append((rows, lo, past + n, b))
            rows += (past + n - lo + 15) // 16 * 16
            self.max_q_len = max(self.max_q_len, n)
        self.rows, self.n_req = rows, len(compact)
        if rows == 0:
            return
        flat = np.concatenate([base, first, np.asarray(compact, dtype=np.int32).T.reshape(-1)]).astype(np.int32)
        host = torch.from_numpy(flat)
        dev = host.pin_memory().to(device, non_blocking=True) if torch.device(device).type == "cuda" else host
        k = self.n_req
        self.row_base, self.first_kv = dev[:B], dev[B:2 * B]
        self.g_base, self.g_first, self.g_len, self.g_req = (dev[2 * B + i * k:2 * B + (i + 1) * k] for i in range(4))


def latent_expand(shape, w_ukv, cache, plan: LatentPlan, block_table, block_size):
    """The cached rows the plan's requests can see as a dense matrix [rows, kv_rank + rot], and their per-head keys and values by one
    product with w_ukv [H * (dim + vdim), kv_rank]."""
    width = shape.R + shape.rot
    lat = torch.empty(plan.rows, width, dtype=torch.bfloat16, device=cache.device)
    _lib.check(_lib.lib().ogb_latent_gather(_ptr(cache), cache.stride(0), _ptr(block_table), block_table.stride(0), int(block_size), _ptr(plan.g_base),
                                           _ptr(plan.g_first), _ptr(plan.g_len), _ptr(plan.g_req), plan.n_req, plan.rows, width, _ptr(lat), width,
                                           _stream()), "latent_gather")
    return lat, linear(lat[:, :shape.R], w_ukv)


def latent_attend_expanded(proj, shape, lat, kv, plan: LatentPlan, cu_seqlens, past_lens, scale, window, out, sinks=None, gate=None):
    """Tensor-memory attention of the plan's requests on expanded keys and values; writes their rows of out [T, >= H * vdim], times the sigmoid
    of gate [T, H * vdim] where one is given (rows of whole 16-byte pieces)."""
    _lib.check(_lib.lib().ogb_attention_tc_latent(_ptr(proj), proj.stride(0), _ptr(kv), kv.stride(0), _ptr(lat), lat.stride(0), shape.R, plan.rows,
                                                 _ptr(cu_seqlens), _ptr(past_lens), _ptr(plan.row_base), _ptr(plan.first_kv), _ptr(out), out.stride(0),
                                                 float(scale), int(window), _ptr(sinks), _ptr(gate), gate.stride(0) if gate is not None else 0,
                                                 past_lens.shape[0], plan.max_q_len, shape.H, shape.dim, shape.rot,
                                                 shape.vdim, workspace(proj.device).status, _stream()), "attention_tc_latent")
    return out


def latent_attention_long(proj, shape, w_ukv, cache, plan: LatentPlan, cu_seqlens, past_lens, block_table, block_size, scale, window, out, sinks=None,
                          gate=None):
    """The long requests of a step (plan): their visible latents are gathered, expanded to keys and values, and attended on the tensor
    cores.  Writes the requests' rows of out [T, >= H * vdim]."""
    lat, kv = latent_expand(shape, w_ukv, cache, plan, block_table, block_size)
    return latent_attend_expanded(proj, shape, lat, kv, plan, cu_seqlens, past_lens, scale, window, out, sinks, gate)


# ------------------------------------------------------------------------------------------ logits processing
def logits_bitmask(logits, mask_words, mask_rows=None):
    if not logits.is_cuda:
        return ref.logits_bitmask(logits, mask_words, mask_rows)
    rows, V = logits.shape
    assert logits.dtype == torch.float32 and logits.is_contiguous() and mask_words.dtype == torch.int32
    _lib.check(_lib.lib().ogb_logits_bitmask(_ptr(logits), rows, V, _ptr(mask_words), _ptr(mask_rows), _stream()), "logits_bitmask")
    return logits


def logits_edit(logits, rows, tokens, ops, values):
    _check_index("logits_edit", "rows", rows, logits.shape[0])
    _check_index("logits_edit", "tokens", tokens, logits.shape[1])
    if not logits.is_cuda:
        return ref.logits_edit(logits, rows, tokens, ops, values)
    assert logits.dtype == torch.float32 and logits.is_contiguous()
    _lib.check(_lib.lib().ogb_logits_edit(_ptr(logits), logits.shape[1], _ptr(rows), _ptr(tokens), _ptr(ops), _ptr(values),
                                          rows.numel(), _stream()), "logits_edit")
    return logits


def to_float32(x):
    if x.dtype == torch.float32:
        return x
    if not x.is_cuda:
        return x.float()
    out = torch.empty(x.shape, dtype=torch.float32, device=x.device)
    _lib.check(_lib.lib().ogb_bf16_to_f32(_ptr(x.contiguous()), _ptr(out), x.numel(), _stream()), "bf16_to_f32")
    return out


def gather_rows(x, rows, f16: bool = False):
    """out[i] = x[rows[i]]; f16: bf16 rows come out as fp16 (input of the fp16 form of the packed FP4 expert GEMM)."""
    _check_index("gather_rows", "rows", rows, x.shape[0])
    if not x.is_cuda:
        return x[rows.long()].to(torch.float16) if f16 else x[rows.long()]
    out = torch.empty(rows.numel(), x.shape[1], dtype=torch.float16 if f16 else x.dtype, device=x.device)
    if f16:
        assert x.dtype == torch.bfloat16
        _lib.check(_lib.lib().ogb_gather_rows_f16(_ptr(x), _ptr(rows), _ptr(out), rows.numel(), x.shape[1] * 2, _stream()), "gather_rows_f16")
        return out
    _lib.check(_lib.lib().ogb_gather_rows(_ptr(x), _ptr(rows), _ptr(out), rows.numel(), x.shape[1] * x.element_size(), _stream()),
               "gather_rows")
    return out


# ------------------------------------------------------------------------------------------ sampling
def _cpu_sample_row(row, k, p, t, seed, pos):
    if k == 1 or t <= 0:
        return int(torch.argmax(row))
    ids, probs = ref.sampled_distribution(row, k if k > 1 else None, p if 0 < p < 1 else None, t)
    rng = np.random.Generator(np.random.Philox(key=int(seed) & ((1 << 64) - 1), counter=[int(pos), 0x5A17, 0, 0]))
    u = rng.random()
    cum = torch.cumsum(probs, 0)
    j = int(torch.searchsorted(cum, torch.tensor(u, dtype=cum.dtype)).clamp(max=len(ids) - 1))
    return int(ids[j])


def sample(logits, top_k, top_p, temperature, seeds, positions, out=None):
    """Per-row sampling.  logits [B, V] fp32; top_k int32 [B] (1 = greedy, <= 0 = no top-k);
    top_p / temperature fp32 [B]; seeds int64 [B]; positions int32 [B] (RNG counter)."""
    B, V = logits.shape
    if not logits.is_cuda:
        res = [_cpu_sample_row(logits[i].float(), int(top_k[i]), float(top_p[i]), float(temperature[i]), int(seeds[i]),
                               int(positions[i])) for i in range(B)]
        return torch.tensor(res, dtype=torch.int32)
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    if out is None:
        out = torch.empty(B, dtype=torch.int32, device=logits.device)
    _lib.check(_lib.lib().ogb_sample(_ptr(logits), logits.stride(0), B, V, _ptr(top_k), _ptr(top_p), _ptr(temperature),
                                     _ptr(seeds), _ptr(positions), _ptr(out), _stream()), "sample")
    return out


def argmax(logits, out=None):
    if not logits.is_cuda:
        return torch.argmax(logits.float(), dim=-1).to(torch.int32)
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    B, V = logits.shape
    if out is None:
        out = torch.empty(B, dtype=torch.int32, device=logits.device)
    _lib.check(_lib.lib().ogb_argmax(_ptr(logits), logits.stride(0), B, V, _ptr(out), _stream()), "argmax")
    return out


def topk(x, k, log_softmax=False, add=None):
    """Sorted top-k per row (k <= 128).  With log_softmax the values are log-probabilities (+ add[row])."""
    if not x.is_cuda:
        return ref.topk(x, k, log_softmax, add)
    assert x.dtype == torch.float32 and x.stride(1) == 1 and k <= 128
    R, n = x.shape
    vals = torch.empty(R, k, dtype=torch.float32, device=x.device)
    idx = torch.empty(R, k, dtype=torch.int32, device=x.device)
    _lib.check(_lib.lib().ogb_topk(_ptr(x), x.stride(0), R, n, k, int(log_softmax), _ptr(add), _ptr(vals), _ptr(idx), _stream()), "topk")
    return vals, idx


def beam_candidates(logits, beam_scores, batch, beams):
    """Beam-search scoring: log-softmax + running beam score, top 2*beams per beam, merged to the best
    2*beams per batch entry.  Returns (scores, tokens, source_beams), each [batch, 2*beams]."""
    cand = 2 * beams
    vals, idx = topk(logits, cand, log_softmax=True, add=beam_scores)
    if not logits.is_cuda:
        v = vals.view(batch, beams * cand)
        order = torch.sort(v, dim=-1, descending=True, stable=True).indices[:, :cand]
        scores = torch.gather(v, 1, order)
        tokens = torch.gather(idx.view(batch, beams * cand), 1, order)
        return scores, tokens.to(torch.int32), (order // cand).to(torch.int32)
    scores = torch.empty(batch, cand, dtype=torch.float32, device=logits.device)
    tokens = torch.empty(batch, cand, dtype=torch.int32, device=logits.device)
    src = torch.empty(batch, cand, dtype=torch.int32, device=logits.device)
    _lib.check(_lib.lib().ogb_beam_merge(_ptr(vals), _ptr(idx), batch, beams, cand, _ptr(scores), _ptr(tokens), _ptr(src), _stream()),
               "beam_merge")
    return scores, tokens, src


_verify_scratch = {}


def verify_sampled(logits, draft, q_dists, top_k: int, top_p: float, temperature: float, seed: int, first_position: int):
    """Sampled speculative verification on the device.  logits [K+1, V] fp32 (target rows for the K draft
    positions and the bonus position); draft: K token ids; q_dists: per draft position None (deterministic
    proposal) or (ids, probs) of the draft model's sampled distribution.  Row i draws with the random stream of
    (seed, first_position + i).  Returns (accepted, commit list, accept probabilities [K])."""
    K = len(draft)
    dev = logits.device
    assert logits.is_cuda and logits.dtype == torch.float32 and logits.shape[0] == K + 1 and 1 < top_k <= 1024
    R = K + 1
    ki = torch.full((R,), int(top_k), dtype=torch.int32, device=dev)
    pp = torch.full((R,), float(top_p), dtype=torch.float32, device=dev)
    tt = torch.full((R,), float(temperature), dtype=torch.float32, device=dev)
    seeds = torch.full((R,), int(seed) & ((1 << 63) - 1), dtype=torch.int64, device=dev)
    pos = torch.arange(first_position, first_position + R, dtype=torch.int32, device=dev)
    d = torch.tensor(list(draft) or [0], dtype=torch.int32, device=dev)
    qs = max([len(q[0]) for q in q_dists if q is not None] + [1])
    qi = np.zeros((max(K, 1), qs), dtype=np.int32)
    qp = np.zeros((max(K, 1), qs), dtype=np.float32)
    qn = np.zeros((max(K, 1),), dtype=np.int32)
    for i, q in enumerate(q_dists):
        if q is not None:
            m = len(q[0])
            qi[i, :m], qp[i, :m], qn[i] = q[0], q[1], m
    qi_d, qp_d, qn_d = torch.from_numpy(qi).to(dev), torch.from_numpy(qp).to(dev), torch.from_numpy(qn).to(dev)
    key = (dev.index, K)
    if key not in _verify_scratch:
        _verify_scratch[key] = torch.zeros(2 * R + 1, dtype=torch.int32, device=dev)
    scratch = _verify_scratch[key]
    out = torch.zeros(R + 2, dtype=torch.int32, device=dev)     # [accepted, status, commit...]
    aprob = torch.zeros(max(K, 1), dtype=torch.float32, device=dev)
    rc = _lib.lib().ogb_verify_sampled(_ptr(logits), logits.stride(0), logits.shape[1], K, _ptr(ki), _ptr(pp), _ptr(tt), _ptr(seeds), _ptr(pos),
                                       _ptr(d), _ptr(qi_d), _ptr(qp_d), _ptr(qn_d), qs, _ptr(scratch), _ptr(aprob), _ptr(out[0:1]),
                                       _ptr(out[2:]), _ptr(out[1:2]), _stream())
    _lib.check(rc, "verify_sampled")
    res = out.tolist()
    if res[1] != 0:
        raise RuntimeError("verify_sampled: sampling parameters outside the device path (needs 1 < top_k <= 1024, temperature > 0)")
    accepted = res[0]
    return accepted, res[2:2 + accepted + 1], aprob[:K].tolist()
