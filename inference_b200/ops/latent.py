"""Latent attention (csrc/kernels/latent_attention.cu): one cached row [c | k_rot] per token serves every head."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .._native import kernels
from .runtime import check, ptr, require_cuda, stream_ptr


def latent_width(rk: int, rot: int) -> int:
    """Columns of a cached row [c | k_rot] with its padding."""
    return rk + (rot + 63) // 64 * 64


@dataclass
class LatentWeights:
    """Sizes and weights of one layer. Projection columns: q (heads x [dn | rp]) or, with q_rank > 0, a query latent (qk) that `uq`
    [heads (dn + rp), qk] takes to q, then the latent (rk), the shared key part (rp), the gate logits (heads). dn, rp, rk, vp are the padded dim, rot_dim, kv_rank and vdim; in the cache the shared key part takes rc
    columns (a multiple of 64, zero beyond rp); padding entries of the weights are zero.
    In the activation type: ukv [heads (dn + vp), rk], the rows of all heads' key projections and then of their value projections
    (uv is the latter part as [heads, vp, rk]), and the transposed key projections uk_t [heads, rk, dn]; norm fp32 [rk], q_norm fp32
    [qk], sink fp32 [heads] or None. window > 0: a query sees only the last `window` keys, its own included."""
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
    sink: torch.Tensor | None
    ukv: torch.Tensor
    uk_t: torch.Tensor
    window: int = 0
    q_rank: int = 0
    qk: int = 0
    q_norm: torch.Tensor | None = None
    uq: torch.Tensor | None = None

    @property
    def uv(self) -> torch.Tensor:
        return self.ukv[self.heads * self.dn:].view(self.heads, self.vp, self.rk)

    @property
    def col_c(self) -> int:
        return self.qk if self.q_rank else self.heads * (self.dn + self.rp)

    @property
    def col_gate(self) -> int:
        return self.col_c + self.rk + self.rp

    @property
    def width(self) -> int:
        """Columns of a cached row."""
        return self.rk + self.rc

    @property
    def rc(self) -> int:
        return latent_width(self.rk, self.rot) - self.rk


@dataclass
class QueryRotation:
    """Rotated query parts that travel with a head product: columns [at, at + rp) of a's head rows (beyond the product's K) are rotated
    (the first `rot` in neighbouring pairs) and stored behind the N columns of out's head rows, rc columns in all."""
    cos: torch.Tensor
    sin: torch.Tensor
    positions: torch.Tensor
    at: int
    rot: int
    rp: int
    rc: int


@dataclass
class SplitPartials:
    """Un-normalised attention results of KV splits: o fp32 [splits, T, heads, rk], ml fp32 [splits, T, heads, 2] (running
    maximum in log2 units, sum of exponentials relative to it)."""
    o: torch.Tensor
    ml: torch.Tensor


def head_product(a: torch.Tensor | SplitPartials, w: torch.Tensor, out: torch.Tensor, *, gate: torch.Tensor | None = None,
                 sink: torch.Tensor | None = None, rows_in: torch.Tensor | None = None,
                 rows_out: torch.Tensor | None = None, rotate: QueryRotation | None = None, kernel: str = "auto") -> torch.Tensor:
    """out[t, h] = w[h] a[t, h], times sigmoid(gate[t, h]). a [T, H, K] and out [T, H, N] strided with unit inner stride, w
    [H, N, K], gate [T, >= H] strided; all in one element type. Split partials as `a` are merged first, exp(sink[h]) joining
    the denominator. rows_in / rows_out int32 [n]: row i is token rows_in[i] of `a`, rows_out[i] of `out` and `gate`. bf16 runs on the MMA kernel (all sizes multiples of 8), fp32 (and
    kernel="simple") on the plain one."""
    merge = isinstance(a, SplitPartials)
    H, N, K = w.shape
    n = next((r.numel() for r in (rows_in, rows_out) if r is not None), out.shape[0])
    require_cuda(w, out, gate, rows_in, rows_out)
    assert out.stride(2) == 1 and w.is_contiguous() and w.dtype == out.dtype and out.shape[1:] == (H, N)
    assert gate is None or (gate.dtype == w.dtype and gate.stride(1) == 1)
    gs = gate.stride(0) if gate is not None else 0
    if w.dtype == torch.bfloat16 and kernel == "auto":
        ap = None if merge else a
        r = rotate
        rot = (None, None, None, 0, 0, 0, 0, 0) if r is None else (r.cos.data_ptr(), r.sin.data_ptr(), r.positions.data_ptr(), r.at, N, r.rot, r.rp, r.rc)
        assert r is None or (r.positions.dtype == torch.int32 and r.cos.dtype == torch.float32 and r.cos.shape[-1] == r.rot // 2)
        assert merge or (a.shape[1:] == (H, K) and a.stride(2) == 1 and a.dtype == w.dtype)
        rc = kernels().swb_head_mma(ptr(ap), ap.stride(0) if ap is not None else 0, ap.stride(1) if ap is not None else 0, w.data_ptr(),
                                    out.data_ptr(), out.stride(0), out.stride(1), ptr(gate), gs, ptr(rows_in),
                                    ptr(rows_out), n, H, N, K, a.o.data_ptr() if merge else None,
                                    a.ml.data_ptr() if merge else None, ptr(sink) if merge else None, a.o.shape[0] if merge else 0,
                                    a.o.shape[1] * H if merge else 0, *rot, stream_ptr())
        check(rc, "swb_head_mma")
        return out
    assert rotate is None
    assert not merge and rows_in is None and rows_out is None and a.shape == (n, H, K) and a.stride(2) == 1 and a.dtype == w.dtype
    rc = kernels().swb_head_product_simple(a.data_ptr(), a.stride(0), a.stride(1), w.data_ptr(), N * K, K, 1, out.data_ptr(),
                                           out.stride(0), out.stride(1), ptr(gate), gs, n, H, N, K,
                                           1 if a.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_head_product_simple")
    return out


def latent_decode_supported(w: LatentWeights, block_size: int) -> bool:
    """Whether the tcgen05 kernel covers the layer (others run on the plain kernel)."""
    return w.rk <= 512 and w.rc <= 128 and w.scale > 0 and block_size % 8 == 0


def latent_decode(q_abs: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, kv_lens: torch.Tensor, w: LatentWeights, *,
                  cu_q: torch.Tensor | None, max_q_len: int, num_splits: int = 1) -> SplitPartials:
    """Causal attention in the latent space on the tcgen05 kernel: q_abs [T, heads, width] bf16 against the cached rows, whose
    leading rk columns are the values."""
    require_cuda(q_abs, cache, block_table, kv_lens)
    T, H, D = q_abs.shape
    assert q_abs.is_contiguous() and cache.is_contiguous() and D == w.width == cache.shape[-1] and q_abs.dtype == torch.bfloat16
    assert block_table.dtype == torch.int32 and kv_lens.dtype == torch.int32 and block_table.stride(1) == 1
    part = SplitPartials(torch.empty((num_splits, T, H, w.rk), dtype=torch.float32, device=q_abs.device),
                         torch.empty((num_splits, T, H, 2), dtype=torch.float32, device=q_abs.device))
    rc = kernels().swb_latent_decode(q_abs.data_ptr(), cache.data_ptr(), cache.shape[0], cache.shape[1], block_table.data_ptr(),
                                     block_table.stride(0), ptr(cu_q), kv_lens.data_ptr(), kv_lens.numel(), max_q_len if cu_q is None else 0, max_q_len,
                                     T, H, w.rk, w.rc, w.rot, w.scale, num_splits, w.window, part.o.data_ptr(), part.ml.data_ptr(), stream_ptr())
    check(rc, "swb_latent_decode")
    return part


def latent_prep(proj: torch.Tensor, w: LatentWeights, eps: float, cos: torch.Tensor, sin: torch.Tensor, positions: torch.Tensor,
                slots: torch.Tensor, cache: torch.Tensor, q_abs: torch.Tensor | None = None,
                q_row: torch.Tensor | None = None) -> None:
    """In place on proj: the latent is normed, the shared key part and the queries' rotated parts are rotated; a query latent is
    normed instead of the queries (they come later, see rotate_queries). [c | k_rot] goes to row `slots` of cache [blocks, block_size,
    width]; q_abs [n, heads, width] receives the rotated query parts at column rk, token t in row q_row[t] (int32 [T], below 0: nowhere;
    null: row t)."""
    require_cuda(proj, cos, sin, positions, slots, cache, q_abs)
    assert proj.stride(1) == 1 and cache.is_contiguous() and cache.shape[-1] == w.width and cache.dtype == proj.dtype
    assert slots.dtype == torch.int64 and positions.dtype == torch.int32 and cos.shape[-1] == w.rot // 2
    low = w.q_rank > 0
    assert not low or q_abs is None
    rc = kernels().swb_latent_prep(None if low else proj.data_ptr(), proj.stride(0), proj.data_ptr(), proj.stride(0), w.col_c,
                                   w.norm.data_ptr(), ptr(w.q_norm), w.q_rank, w.qk, eps, cos.data_ptr(), sin.data_ptr(),
                                   positions.data_ptr(), slots.data_ptr(), cache.data_ptr(), ptr(q_abs), ptr(q_row), proj.shape[0],
                                   0 if low else w.heads, w.dn, w.rot, w.rp, w.rc, w.rank, w.rk, 1 if proj.dtype == torch.float32 else 0,
                                   stream_ptr())
    check(rc, "swb_latent_prep")


def rotate_queries(q: torch.Tensor, w: LatentWeights, cos: torch.Tensor, sin: torch.Tensor, positions: torch.Tensor,
                   q_abs: torch.Tensor | None = None, q_row: torch.Tensor | None = None) -> None:
    """The rotated parts of q [T, heads * (dn + rp)], in place and (q_abs, q_row as in latent_prep) into the latent-space queries."""
    require_cuda(q, cos, sin, positions, q_abs, q_row)
    assert q.stride(1) == 1 and positions.dtype == torch.int32 and cos.shape[-1] == w.rot // 2
    assert q_abs is None or q_abs.dtype == q.dtype
    rc = kernels().swb_latent_prep(q.data_ptr(), q.stride(0), None, 0, 0, None, None, 0, 0, 0.0, cos.data_ptr(), sin.data_ptr(),
                                   positions.data_ptr(), None, None, ptr(q_abs), ptr(q_row), q.shape[0], w.heads, w.dn, w.rot, w.rp, w.rc,
                                   w.rank, w.rk, 1 if q.dtype == torch.float32 else 0, stream_ptr())
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
                                   kv_lens.data_ptr(), kv_lens.numel(), max_q_len, T, H, 1, D, w.rk, D, w.scale, 0, ptr(w.sink), w.window, 0.0, None, 1,
                                   0, None, 0,
                                   1 if q_abs.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_attn_simple")
    return out


def latent_prefill_supported(w: LatentWeights) -> bool:
    """Whether the tcgen05 prefill kernel on expanded keys and values covers the layer."""
    return w.dn <= 128 and w.rp <= 64 and w.vp <= 128 and w.scale > 0


def latent_gather(cache: torch.Tensor, block_table: torch.Tensor, cu_k: torch.Tensor, rows: int,
                  seqs: torch.Tensor | None = None, first: torch.Tensor | None = None) -> torch.Tensor:
    """The cached rows of several sequences side by side [rows, width]: sequence seqs[i] (null: i) of the block table, from its row
    first[i] (int32, null: 0) on, at [cu_k[i], cu_k[i + 1]), cu_k int32 on the device, rows = its last entry."""
    require_cuda(cache, block_table, cu_k, seqs, first)
    width = cache.shape[-1]
    assert cache.is_contiguous() and cache.dtype == torch.bfloat16 and cu_k.dtype == torch.int32
    out = torch.empty((rows, width), dtype=cache.dtype, device=cache.device)
    rc = kernels().swb_latent_gather(cache.data_ptr(), block_table.data_ptr(), block_table.stride(0), cache.shape[1], ptr(seqs), ptr(first),
                                     cu_k.data_ptr(), cu_k.numel() - 1, rows, width, out.data_ptr(), stream_ptr())
    check(rc, "swb_latent_gather")
    return out


def latent_prefill(q: torch.Tensor, kv: torch.Tensor, k_rot: torch.Tensor, w: LatentWeights, out: torch.Tensor, *, cu_q: torch.Tensor,
                   max_q_len: int, gate: torch.Tensor | None = None, seqs: torch.Tensor | None = None,
                   cu_k: torch.Tensor | None = None) -> torch.Tensor:
    """Causal attention on expanded keys and values (tcgen05 kernel, bf16). q [T, heads * (dn + rp)] strided rows, kv [R, heads *
    (dn + vp)] (all keys, then all values), k_rot [R, rp] strided rows, gate [T, >= heads] logits, out [T, heads * vp]. seqs int32
    [n]: only these sequences of cu_q (null: all); cu_k int32 [n + 1]: their key rows, the last of them those of the queries
    (null: R = T, the queries' own rows). A window
    counts from the end, so key rows in front of every query's window need not be there."""
    require_cuda(q, kv, k_rot, out, cu_q, gate, seqs, cu_k)
    assert q.stride(1) == 1 and kv.stride(1) == 1 and k_rot.stride(1) == 1 and out.stride(1) == 1
    assert all(t.dtype == torch.bfloat16 for t in (q, kv, k_rot, out)) and kv.shape[1] == w.heads * (w.dn + w.vp)
    assert gate is None or (gate.dtype == torch.bfloat16 and gate.stride(1) == 1)
    n = seqs.numel() if seqs is not None else cu_q.numel() - 1
    assert cu_k is None or cu_k.numel() == n + 1
    rc = kernels().swb_latent_prefill(q.data_ptr(), q.stride(0), kv.data_ptr(), kv[:, w.heads * w.dn:].data_ptr(), kv.stride(0),
                                      k_rot.data_ptr(), k_rot.stride(0), kv.shape[0], out.data_ptr(), out.stride(0), n, max_q_len,
                                      q.shape[0], w.heads, w.dn, w.rp, w.vp, w.scale, ptr(w.sink), ptr(gate),
                                      gate.stride(0) if gate is not None else 0, cu_q.data_ptr(), ptr(seqs), ptr(cu_k), w.window, stream_ptr())
    check(rc, "swb_latent_prefill")
    return out
