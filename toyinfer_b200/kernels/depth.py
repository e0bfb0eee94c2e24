"""A float32 residual stream that is averaged over depth, the norm that reads it and the token shift (csrc/depth_stream.cu)."""
from __future__ import annotations

from ctypes import c_float, c_int, c_void_p
from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from . import KernelError, _call, _i32, _need_cuda, _ptr, _stream
from .wide import _fn

P, I, F = c_void_p, c_int, c_float
MAX_RESULTS = 256


@dataclass
class DepthUpdate:
    """What a layer left pending on a stream whose history is ``results`` = [X_0 .. X_n-1] (float32 [M, H] each): the layer
    read y = sum_j average_in[j] X_j (None: the last result) and its result is X_n = y + mult * (first + second); what goes
    on is sum_{j <= n} average_out[j] X_j (None: X_n)."""

    results: List[torch.Tensor]
    first: torch.Tensor                             # [M, H], the engine's type
    second: Optional[torch.Tensor] = None
    mult: float = 1.0
    average_in: Optional[torch.Tensor] = None       # float32 [n]
    average_out: Optional[torch.Tensor] = None      # float32 [n + 1]


@dataclass
class ShiftedRead:
    """The token shift of a read: z'_t = z_t + (z_{t-1} - z_t) * mix, with the last z of every sequence in ``state``
    (float32 [slots, H], zero when the sequence starts)."""

    mix: torch.Tensor                               # float32 [H]
    state: torch.Tensor
    batch: object


def _f32(t: Optional[torch.Tensor], shape, what: str) -> None:
    if t is not None and (t.dtype != torch.float32 or tuple(t.shape) != tuple(shape) or not t.is_contiguous()):
        raise KernelError(f"depth_norm: {what} must be dense float32 {tuple(shape)}, got {t.dtype} {tuple(t.shape)}")


def depth_norm(x0: torch.Tensor, pending: Optional[DepthUpdate], weight: Optional[torch.Tensor], eps: float, out_dtype: torch.dtype,
               shift: Optional[ShiftedRead] = None, rows: Optional[torch.Tensor] = None, want_sum: bool = False):
    """Reads the stream after the pending layer (none: x0 [M, H] itself) -> (z, z', results, sum): z = rmsnorm(y) * weight in
    ``out_dtype`` (None without a weight), z' the same after the token shift (None without ``shift``), results the history
    with the pending layer's result written at its end, sum the float32 y with ``want_sum``.  With ``rows`` only those rows
    are formed, and no result is written."""
    results = pending.results if pending is not None else [x0]
    first = pending.first if pending is not None else None
    second = pending.second if pending is not None else None
    c_in = pending.average_in if pending is not None else None
    c_out = pending.average_out if pending is not None else None
    _need_cuda(*results, first, second, c_in, c_out, weight, rows, what="depth_norm")
    M, H = x0.shape
    n = len(results)
    if n > MAX_RESULTS:
        raise KernelError(f"depth_norm: a history of {n} results is not supported (up to {MAX_RESULTS})")
    for X in results:
        _f32(X, (M, H), "a layer's result")
    for y in (first, second):
        if y is not None and (tuple(y.shape) != (M, H) or y.dtype != out_dtype or not y.is_contiguous()):
            raise KernelError(f"depth_norm: a pending output must be dense {out_dtype} [{M}, {H}]")
    _f32(c_in, (n,), "the coefficients of the layer's input")
    _f32(c_out, (n + 1,), "the coefficients of what goes on")
    _f32(weight, (H,), "the norm weight")
    R, x_out = M, None
    if rows is not None:
        _i32(rows, "depth_norm rows")
        R = rows.numel()
        if shift is not None:
            raise KernelError("depth_norm: gathered rows take no shift")
    elif pending is not None:
        x_out = torch.empty((M, H), dtype=torch.float32, device=x0.device)
    out = torch.empty((R, H), dtype=out_dtype, device=x0.device) if weight is not None else None
    total = torch.empty((R, H), dtype=torch.float32, device=x0.device) if want_sum else None
    mix = shifted = prev = state = tok_seq = seq_slot = cu_new = None
    by_slot = one_each = 0
    if shift is not None:
        b = shift.batch
        mix, state = shift.mix, shift.state
        _f32(mix, (H,), "the shift")
        if state.dtype != torch.float32 or state.dim() != 2 or state.shape[1] != H or not state.is_contiguous():
            raise KernelError(f"depth_norm: the shift's state must be dense float32 [slots, {H}]")
        shifted = torch.empty((R, H), dtype=out_dtype, device=x0.device)
        tok_seq, seq_slot, cu_new = b.tok_seq, b.seq_slot, b.cu_new
        if b.mode == "extend":                 # a row is a sequence: the block that reads its state is the one that writes it
            prev, by_slot, one_each = state, 1, 1
        elif b.mode != "start":                # a sequence's rows may lie in several blocks: its state is read from a copy
            from . import gather_add
            prev = gather_add(state, None, seq_slot)
    ptrs = (c_void_p * n)(*[X.data_ptr() for X in results])
    _call(_fn("ti_depth_norm", [P, I, P, P, P, P, F, P, P, F, P, P, P, P, P, I, P, P, P, P, P, I, I, I, I, I, P]),
          ptrs, n, _ptr(c_in), _ptr(c_out), _ptr(first), _ptr(second), float(pending.mult) if pending is not None else 1.0, _ptr(x_out),
          _ptr(weight), float(eps), _ptr(out), _ptr(total), _ptr(mix), _ptr(shifted), _ptr(prev), by_slot, _ptr(state), _ptr(tok_seq),
          _ptr(seq_slot), _ptr(cu_new), _ptr(rows), R, H, M, one_each, 0 if out_dtype == torch.float32 else 1, _stream())
    if x_out is not None:
        # without averaging nothing reads the older results again
        results = results + [x_out] if c_out is not None else [x_out]
    return out, shifted, results, total
