"""Wrappers of the kernels around several residual streams and the short convolution of a sublayer's input (csrc/kernels/hyper_stream.cu)."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .._native import kernels
from .runtime import check, ptr, require_cuda, stream_ptr
from .stream import NormWeights, RoutedRows

MAX_STREAMS, MAX_WIDTH = 16, 16384


@dataclass
class StreamMix:
    """How a sublayer's result joins the streams: mix fp32 [S (from), S (to)], put fp32 [S]."""
    mix: torch.Tensor
    put: torch.Tensor


@dataclass
class HyperBranch:
    """A sublayer's result: rows `y`; or, with norms, N(y) w_y + N(y2) w_y2 (RMS norms); or weighted expert rows."""
    y: torch.Tensor | RoutedRows
    norm: NormWeights | None = None
    y2: torch.Tensor | None = None
    norm2: NormWeights | None = None


@dataclass
class ShortConv:
    """A causal convolution over time on every channel, added to its input. w fp32 [taps, Hp], the last row the current token's; window
    [slots, taps - 1, Hp] in the activation type: the inputs in front of the step, moved on by the convolution."""
    w: torch.Tensor
    window: torch.Tensor

    @property
    def taps(self) -> int:
        return self.w.shape[0]


def _check_conv(conv: ShortConv, h: torch.Tensor, slots: torch.Tensor, positions: torch.Tensor) -> None:
    Hp = h.shape[1]
    assert conv.w.dtype == torch.float32 and conv.w.is_contiguous() and conv.w.shape[1] == Hp
    assert conv.window.dtype == h.dtype and conv.window.is_contiguous() and conv.window.shape[1:] == (conv.taps - 1, Hp)
    assert slots.dtype == torch.int32 and positions.dtype == torch.int32


def hyper_step(x: torch.Tensor, streams: int, width: int, eps: float, *, branch: HyperBranch | None = None, join: StreamMix | None = None,
               x_out: torch.Tensor | None = None, read: torch.Tensor | None = None, norm: NormWeights | None = None,
               out: torch.Tensor | None = None, rows: torch.Tensor | None = None, conv: ShortConv | None = None,
               slots: torch.Tensor | None = None, positions: torch.Tensor | None = None) -> torch.Tensor | None:
    """With a branch y: x_t <- sum_s mix[s, t] x_s + put[t] y for all streams t at once. Then, with `out`: out = N(sum_t read[t] x_t) w, the
    RMS norm over `width` columns (read fp32 [S], None: the plain sum), and with `conv` h + conv(h) of that h, for steps of one token per
    sequence (slots int32 [T], below 0: no window; positions int32 [T], 0: starts from zeros).

    x fp32 [T, S, Hp], or [T, Hp] when all streams are still alike; the joined streams go to x_out [T, S, Hp] (x itself may be it). rows
    int64 [R]: only these tokens are normed (no branch)."""
    require_cuda(x, out, x_out, read, rows)
    assert x.dtype == torch.float32 and x.stride(-1) == 1
    T, Hp = x.shape[0], x.shape[-1]
    in_tok, in_stream = x.stride(0), x.stride(1) if x.dim() == 3 else 0
    assert x.dim() == 2 or x.shape[1] == streams
    b, E = branch, None
    y = pick = weights = None
    if b is not None:
        y = b.y.y if isinstance(b.y, RoutedRows) else b.y
        E = y.dtype
        assert join is not None and x_out is not None and x_out.shape == (T, streams, Hp) and x_out.is_contiguous() and x_out.dtype == torch.float32
        assert join.mix.shape == (streams, streams) and join.mix.is_contiguous() and join.put.numel() == streams
        assert join.mix.dtype == join.put.dtype == torch.float32 and y.stride(1) == 1 and y.shape[1] == Hp
        if isinstance(b.y, RoutedRows):
            pick, weights = b.y.rows, b.y.weights
            assert pick.shape == weights.shape and pick.shape[0] == T and pick.dtype == torch.int32 and weights.dtype == torch.float32
            assert pick.is_contiguous() and weights.is_contiguous()
        else:
            assert y.shape[0] == T
        assert b.y2 is None or (b.y2.shape == (T, Hp) and b.y2.dtype == E and b.y2.stride(1) == 1 and b.norm is not None and b.norm2 is not None)
    for n in (norm, b.norm if b else None, b.norm2 if b else None):
        assert n is None or (n.w.dtype == torch.float32 and n.w.numel() == Hp and n.w.is_contiguous() and n.b is None)
    if out is not None:
        assert norm is not None and out.stride(1) == 1 and out.shape == ((rows.numel() if rows is not None else T), Hp) and E in (None, out.dtype)
        E = out.dtype
    assert E in (torch.bfloat16, torch.float32) and (read is None or (read.dtype == torch.float32 and read.numel() == streams))
    if conv is not None:
        _check_conv(conv, out, slots, positions)
        assert slots.numel() == T == positions.numel()
    n_rows = rows.numel() if rows is not None else T
    dims = (ctypes.c_int * 8)(n_rows, streams, width, Hp, pick.shape[1] if pick is not None else 0, conv.taps if conv is not None else 1,
                              1 if E == torch.float32 else 0, slots.numel() if conv is not None else 0)
    rc = kernels().swb_hyper_step(
        dims, x.data_ptr(), in_tok, in_stream, ptr(x_out), ptr(rows), ptr(join.mix) if join is not None else None,
        ptr(join.put) if join is not None else None, ptr(read), ptr(y), y.stride(0) if y is not None else 0,
        ptr(b.norm.w) if b is not None and b.norm is not None else None, ptr(b.y2) if b is not None else None,
        b.y2.stride(0) if b is not None and b.y2 is not None else 0, ptr(b.norm2.w) if b is not None and b.norm2 is not None else None,
        ptr(pick), ptr(weights), ptr(norm.w) if norm is not None else None, ptr(out), out.stride(0) if out is not None else 0, eps,
        ptr(conv.w) if conv is not None else None, ptr(conv.window) if conv is not None else None, ptr(slots) if conv is not None else None,
        ptr(positions) if conv is not None else None, stream_ptr())
    check(rc, "swb_hyper_step")
    return out


def short_conv(h: torch.Tensor, conv: ShortConv, slots: torch.Tensor, positions: torch.Tensor, *, cu_q: torch.Tensor | None,
               max_q_len: int) -> torch.Tensor:
    """h + conv(h) over a ragged batch: slots int32 [num_seqs], positions int32 [T], cu_q int32 [num_seqs + 1] or None (max_q_len tokens
    each). h [T, Hp] in bf16 or fp32."""
    require_cuda(h, conv.w, conv.window, slots, positions, cu_q)
    assert h.stride(1) == 1 and h.dtype in (torch.bfloat16, torch.float32)
    _check_conv(conv, h, slots, positions)
    out = torch.empty(h.shape, dtype=h.dtype, device=h.device)
    rc = kernels().swb_short_conv(h.data_ptr(), h.stride(0), out.data_ptr(), out.stride(0), conv.w.data_ptr(), conv.taps, conv.window.data_ptr(),
                                  slots.data_ptr(), positions.data_ptr(), ptr(cu_q), slots.numel(), max_q_len, h.shape[1],
                                  1 if h.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_short_conv")
    return out
