"""Latent attention (csrc/kernels/latent_attention.cu): one cached row [c | k_rot] per token serves every head."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .._native import kernels
from .runtime import check, ptr, require_cuda, stream_ptr


@dataclass
class LatentWeights:
    """Sizes and weights of one layer. Projection columns: q (heads x [dn | rp]), the latent (rk), the shared key part (rp), the
    gate logits (heads). dn, rp, rk, vp are the padded dim, rot_dim, kv_rank and vdim; padding entries of the weights are zero.
    uk [heads, dn, rk] and uv [heads, vp, rk] in the activation type, norm fp32 [rk], sink fp32 [heads]."""
    heads: int
    dim: int
    dn: int
    rot: int
    rp: int
    rank: int
    rk: int
    vdim: int
    vp: int
    scale: float
    norm: torch.Tensor
    sink: torch.Tensor
    uk: torch.Tensor
    uv: torch.Tensor

    @property
    def col_c(self) -> int:
        return self.heads * (self.dn + self.rp)

    @property
    def col_gate(self) -> int:
        return self.col_c + self.rk + self.rp

    @property
    def width(self) -> int:
        return self.rk + self.rp


def head_product(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, *, transpose: bool = False,
                 gate: torch.Tensor | None = None) -> torch.Tensor:
    """out[t, h] = w[h] a[t, h] (w[h]^T with `transpose`), times sigmoid(gate[t, h]). a [T, H, K] and out [T, H, N] strided
    with unit inner stride, w [H, N, K] (or [H, K, N]), gate [T, H] strided; all in one element type."""
    require_cuda(a, w, out)
    T, H, K = a.shape
    N = out.shape[2]
    assert a.stride(2) == 1 and out.stride(2) == 1 and w.is_contiguous() and a.dtype == w.dtype == out.dtype
    assert w.shape == ((H, K, N) if transpose else (H, N, K)) and (gate is None or (gate.dtype == a.dtype and gate.stride(1) == 1))
    rc = kernels().swb_head_product_simple(a.data_ptr(), a.stride(0), a.stride(1), w.data_ptr(), N * K, 1 if transpose else K,
                                           N if transpose else 1, out.data_ptr(), out.stride(0), out.stride(1), ptr(gate),
                                           gate.stride(0) if gate is not None else 0, T, H, N, K,
                                           1 if a.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_head_product_simple")
    return out


def latent_prep(proj: torch.Tensor, w: LatentWeights, eps: float, cos: torch.Tensor, sin: torch.Tensor, positions: torch.Tensor,
                slots: torch.Tensor, cache: torch.Tensor, q_abs: torch.Tensor | None = None) -> None:
    """In place on proj: the latent is normed, the shared key part and the queries' rotated parts are rotated. [c | k_rot]
    goes to row `slots` of cache [blocks, block_size, width]; q_abs [T, heads, width] receives the rotated query parts at
    column rk."""
    require_cuda(proj, cos, sin, positions, slots, cache, q_abs)
    assert proj.stride(1) == 1 and cache.is_contiguous() and cache.shape[-1] == w.width and cache.dtype == proj.dtype
    assert slots.dtype == torch.int64 and positions.dtype == torch.int32 and cos.shape[-1] == w.rot // 2
    rc = kernels().swb_latent_prep(proj.data_ptr(), proj.stride(0), w.col_c, w.norm.data_ptr(), eps, cos.data_ptr(), sin.data_ptr(),
                                   positions.data_ptr(), slots.data_ptr(), cache.data_ptr(), ptr(q_abs), proj.shape[0], w.heads,
                                   w.dn, w.rot, w.rp, w.rank, w.rk, 1 if proj.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_latent_prep")


def latent_attention_simple(q_abs: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, kv_lens: torch.Tensor,
                            w: LatentWeights, *, cu_q: torch.Tensor | None, max_q_len: int) -> torch.Tensor:
    """Causal attention in the latent space on the plain fp32-arithmetic kernel: q_abs [T, heads, width] against the cached rows,
    whose leading rk columns are the values -> [T, heads, rk]."""
    require_cuda(q_abs, cache, block_table, kv_lens)
    T, H, D = q_abs.shape
    out = torch.empty((T, H, w.rk), dtype=q_abs.dtype, device=q_abs.device)
    rc = kernels().swb_attn_simple(q_abs.data_ptr(), q_abs.stride(0), cache.data_ptr(), cache.data_ptr(), out.data_ptr(),
                                   out.stride(0), block_table.data_ptr(), block_table.stride(0), cache.shape[1], ptr(cu_q),
                                   kv_lens.data_ptr(), kv_lens.numel(), max_q_len, T, H, 1, D, w.rk, D, w.scale, 0, w.sink.data_ptr(),
                                   1 if q_abs.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_attn_simple")
    return out
