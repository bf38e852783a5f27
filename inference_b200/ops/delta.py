"""Gated delta rule with a decay per key channel or per head (csrc/kernels/delta_rule.cu)."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .._native import kernels
from .runtime import check, ptr, require_cuda, stream_ptr

_WIDTHS = (32, 64, 96, 128, 192, 256, 512)


def delta_key_width(dim: int) -> int | None:
    """Padded key width the recurrence runs at, None above the widest one."""
    return next((w for w in _WIDTHS if w >= dim), None)


@dataclass
class DeltaWeights:
    """Sizes and small tensors of one layer. Projection columns: q [kv_heads * dp], k, v [heads * vp], then (from col_b on)
    one step-size logit per head; with one decay per head (head_decay) its logits stand in the same projection from col_a on; conv fp32 [taps, 2 kv_heads dp + heads vp] in the same order; a_log fp32 [heads], dt_bias fp32
    [heads * dp] ([heads] with head_decay), norm fp32 [vp]; padding entries are zero."""
    heads: int
    kv_heads: int
    dim: int
    dp: int
    vdim: int
    vp: int
    col_b: int
    conv: torch.Tensor
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    norm: torch.Tensor
    head_decay: bool = False
    col_a: int = 0

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dp + self.heads * self.vp

    @property
    def taps(self) -> int:
        return self.conv.shape[0]

    def state_shape(self) -> tuple[int, ...]:
        return (self.heads, self.vp, self.dp)

    def window_shape(self) -> tuple[int, ...]:
        return (self.taps - 1, self.channels)


def channel_delta(proj: torch.Tensor, decay: torch.Tensor, gate: torch.Tensor, w: DeltaWeights, eps: float, state: torch.Tensor,
                  window: torch.Tensor, slots: torch.Tensor, positions: torch.Tensor, *, cu_q: torch.Tensor | None,
                  max_q_len: int) -> torch.Tensor:
    """Short convolutions, the recurrence from the states in `slots` (int32 [num_seqs], below 0: none), output norm and gate.

    proj [T, >= col_b + heads], decay [T, heads * dp] (logits of the decay before softplus), gate [T, heads * vp] (logits), all
    in the activation type; state fp32 [slots, heads, vp, dp] and window [slots, taps - 1, channels] move on in place.
    positions int32 [T]: a sequence that starts this step at position 0 starts from zero. -> [T, heads * vp]."""
    assert not w.head_decay
    return _delta(proj, decay, gate, w, eps, state, window, slots, positions, cu_q, max_q_len, False)


def head_delta(proj: torch.Tensor, gate: torch.Tensor, w: DeltaWeights, eps: float, state: torch.Tensor, window: torch.Tensor,
               slots: torch.Tensor, positions: torch.Tensor, *, cu_q: torch.Tensor | None, max_q_len: int) -> torch.Tensor:
    """As channel_delta with one decay per head, whose logits are columns col_a .. of proj, and a gate that is silu of its logits."""
    assert w.head_decay and proj.shape[1] >= w.col_a + w.heads
    return _delta(proj, proj[:, w.col_a:w.col_a + w.heads], gate, w, eps, state, window, slots, positions, cu_q, max_q_len, True)


def _delta(proj, decay, gate, w: DeltaWeights, eps: float, state, window, slots, positions, cu_q, max_q_len: int, gate_silu: bool) -> torch.Tensor:
    require_cuda(proj, decay, gate, state, window, slots, positions)
    T, S = proj.shape[0], slots.numel()
    E, dev = proj.dtype, proj.device
    assert E in (torch.bfloat16, torch.float32) and decay.dtype == E and gate.dtype == E and window.dtype == E
    assert proj.stride(1) == 1 and decay.stride(1) == 1 and gate.stride(1) == 1 and state.is_contiguous() and window.is_contiguous()
    assert state.dtype == torch.float32 and state.shape[1:] == w.state_shape() and window.shape[1:] == w.window_shape()
    assert slots.dtype == torch.int32 and positions.dtype == torch.int32 and proj.shape[1] >= w.col_b + w.heads
    dims = (ctypes.c_int * 11)(T, S, max_q_len, w.heads, w.kv_heads, w.dim, w.dp, w.vdim, w.vp, w.taps, 1 if w.head_decay else 0)
    common = (dims, ptr(cu_q), positions.data_ptr(), slots.data_ptr())
    fp32 = 1 if E == torch.float32 else 0

    def buf(*shape: int) -> torch.Tensor:
        return torch.empty(shape, dtype=torch.float32, device=dev)
    qk, kq, beta = buf(T, w.kv_heads, 2, w.dp), buf(T, w.kv_heads), buf(T, w.heads)
    g, v, o = buf(T, w.heads, *(() if w.head_decay else (w.dp,))), buf(T, w.heads, w.vp), buf(T, w.heads, w.vp)
    check(kernels().swb_delta_prep(*common, proj.data_ptr(), proj.stride(0), w.col_b, decay.data_ptr(), decay.stride(0),
                                   w.conv.data_ptr(), window.data_ptr(), w.a_log.data_ptr(), w.dt_bias.data_ptr(), qk.data_ptr(),
                                   kq.data_ptr(), g.data_ptr(), v.data_ptr(), beta.data_ptr(), fp32, stream_ptr()), "swb_delta_prep")
    check(kernels().swb_delta_scan(*common, qk.data_ptr(), kq.data_ptr(), g.data_ptr(), v.data_ptr(), beta.data_ptr(),
                                   state.data_ptr(), o.data_ptr(), stream_ptr()), "swb_delta_scan")
    out = torch.empty((T, w.heads * w.vp), dtype=E, device=dev)
    check(kernels().swb_delta_post(*common, o.data_ptr(), gate.data_ptr(), gate.stride(0), w.norm.data_ptr(), eps, 1 if gate_silu else 0, out.data_ptr(),
                                   proj.data_ptr(), proj.stride(0), window.data_ptr(), fp32, stream_ptr()), "swb_delta_post")
    return out
