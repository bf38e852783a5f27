"""Wrappers of the kernels around a 32-bit residual stream (csrc/kernels/stream_ops.cu)."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .._native import kernels
from .runtime import check, ptr, require_cuda, stream_ptr


@dataclass
class NormWeights:
    """A norm's fp32 weight and optional bias, padded with zeros to the padded row width."""
    w: torch.Tensor
    b: torch.Tensor | None = None


@dataclass
class RoutedRows:
    """Expert outputs: token t gets the sum over k of weights[t, k] y[rows[t, k]]; rows int32, weights fp32, both [T, top]."""
    y: torch.Tensor
    rows: torch.Tensor
    weights: torch.Tensor


@dataclass
class Branch:
    """A sublayer output that has not joined the stream yet: rows [*, Hp] in bf16 / fp32, normed on the way in. With
    `rows` (int32 [T, top]) the branch of token t is the sum of y[rows[t, k]] over k times `weight`. `extra` is added to it."""
    y: torch.Tensor
    norm: NormWeights | None
    rows: torch.Tensor | None = None
    top: int = 1
    weight: float = 1.0
    extra: RoutedRows | None = None


@dataclass
class DepthAverage:
    """Results of the earlier layers: fp32 [slots, T, Hp], `filled` of them written; weights fp32 [filled + 1]."""
    results: torch.Tensor
    filled: int
    weights: torch.Tensor


def stream_norm(x: torch.Tensor, width: int, eps: float, *, branch: Branch | None = None, norm: NormWeights | None = None,
                out: torch.Tensor | None = None, out_rows: torch.Tensor | None = None, out_top: int = 1,
                rows: torch.Tensor | None = None, center: bool = True, out_scale: float = 1.0, groups: int = 1,
                x_in: torch.Tensor | None = None, average: DepthAverage | None = None) -> torch.Tensor | None:
    """x += norm(branch); out = norm(x) * out_scale (x itself without `norm`). x fp32 [T, Hp] (in place), `width` <= Hp real
    columns, out bf16 / fp32 rows. out_rows int32 [T, out_top]: the row is stored at all of these rows of `out`. rows
    int64 [R]: only these rows of x are normed (no branch). center: layer norm (mean removed), else RMS norm, over each of `groups` equal
    parts of the row on its own. x_in: the stream is read from there (same layout) and the sum goes to x. average: the sum is
    filed as the next of `results`, and x (and what `out` sees) becomes the weighted sum of all of them."""
    require_cuda(x, out, x_in)
    Hp = x.shape[1]
    T = rows.numel() if rows is not None else x.shape[0]
    assert x.dtype == torch.float32 and x.stride(1) == 1
    b, w1, w2 = branch, (branch.norm if branch is not None else None), norm
    ex = b.extra if b is not None else None
    if ex is not None:
        assert ex.rows.dtype == torch.int32 and ex.weights.dtype == torch.float32 and ex.rows.is_contiguous() and ex.weights.is_contiguous()
        assert ex.rows.shape == ex.weights.shape and ex.rows.shape[0] == T
    for t in (b.y if b is not None else None, out, ex.y if ex is not None else None):
        assert t is None or (t.stride(1) == 1 and t.shape[1] == Hp and t.dtype in (torch.bfloat16, torch.float32))
    for n in (w1, w2):
        assert n is None or (n.w.dtype == torch.float32 and n.w.numel() == Hp and n.w.is_contiguous())
    assert x_in is None or (x_in.dtype == torch.float32 and x_in.stride() == x.stride() and x_in.shape == x.shape)
    av = average
    if av is not None:
        assert b is not None and av.results.dtype == torch.float32 and av.results.shape[1:] == x.shape and av.results.stride()[1:] == x.stride()
        assert av.filled < av.results.shape[0] and av.weights.numel() == av.filled + 1 and av.weights.dtype == torch.float32
    rc = kernels().swb_stream_norm(
        x.data_ptr(), x.stride(0), ptr(rows), ptr(b.y) if b is not None else None, b.y.stride(0) if b is not None else 0,
        1 if b is not None and b.y.dtype == torch.float32 else 0, ptr(b.rows) if b is not None else None,
        b.top if b is not None else 0, b.weight if b is not None else 1.0, ptr(w1.w) if w1 is not None else None,
        ptr(w1.b) if w1 is not None else None, ptr(w2.w) if w2 is not None else None, ptr(w2.b) if w2 is not None else None,
        ptr(out), out.stride(0) if out is not None else 0, 1 if out is not None and out.dtype == torch.float32 else 0,
        ptr(out_rows), out_top, T, width, Hp, eps, out_scale, 1 if center else 0, groups, ptr(x_in),
        ptr(av.results) if av is not None else None, av.results.stride(0) if av is not None else 0, av.filled if av is not None else 0,
        ptr(av.weights) if av is not None else None, ptr(ex.y) if ex is not None else None, ex.y.stride(0) if ex is not None else 0,
        1 if ex is not None and ex.y.dtype == torch.float32 else 0, ptr(ex.rows) if ex is not None else None,
        ptr(ex.weights) if ex is not None else None, ex.rows.shape[1] if ex is not None else 0, stream_ptr())
    check(rc, "swb_stream_norm")
    return out


def stream_embed(ids: torch.Tensor, table: torch.Tensor, *, copies: list[torch.Tensor] | None = None, scale: float = 1.0,
                 out: torch.Tensor | None = None) -> torch.Tensor:
    """fp32 rows of `table` [vocab, Hp] for int64 ids, times `scale`; `copies` (at most two, strided [T, Hp] views in the activation type)
    receive the same rows."""
    require_cuda(ids, table)
    assert ids.dtype == torch.int64 and table.is_contiguous()
    flat = ids.reshape(-1)
    T, Hp = flat.numel(), table.shape[1]
    x = torch.empty((T, Hp), dtype=torch.float32, device=table.device) if out is None else out
    assert x.shape == (T, Hp) and x.is_contiguous() and x.dtype == torch.float32
    c = list(copies or [])
    assert len(c) <= 2 and all(t.stride(1) == 1 and t.shape == (T, Hp) and t.dtype == c[0].dtype for t in c)
    c += [None] * (2 - len(c))
    rc = kernels().swb_stream_embed(flat.data_ptr(), table.data_ptr(), 1 if table.dtype == torch.float32 else 0,
                                    table.shape[0], x.data_ptr(), Hp, ptr(c[0]), c[0].stride(0) if c[0] is not None else 0,
                                    ptr(c[1]), c[1].stride(0) if c[1] is not None else 0,
                                    1 if c[0] is not None and c[0].dtype == torch.float32 else 0, scale, T, Hp,
                                    stream_ptr())
    check(rc, "swb_stream_embed")
    return x


def stream_embed_pairs(ids: torch.Tensor, table: torch.Tensor, pairs: torch.Tensor, mul_prev: int, mul_cur: int, *, positions: torch.Tensor,
                       slots: torch.Tensor, tokens: torch.Tensor, block_table: torch.Tensor, cu_q: torch.Tensor | None, num_seqs: int,
                       max_q_len: int) -> torch.Tensor:
    """fp32 rows table[id] + pairs[(previous id * mul_prev + id * mul_cur) mod buckets]; a sequence's first token takes the last row
    of `pairs` [buckets + 1, Hp]. tokens int32 [blocks, block_size]: paged cache of the ids, in which every token files its own and
    the first token of a sequence in this step finds its predecessor."""
    require_cuda(ids, table, pairs, positions, slots, tokens, block_table, cu_q)
    assert ids.dtype == torch.int64 and table.is_contiguous() and pairs.is_contiguous() and table.dtype == pairs.dtype
    assert positions.dtype == torch.int32 and slots.dtype == torch.int64 and tokens.dtype == torch.int32 and tokens.is_contiguous()
    assert block_table.dtype == torch.int32 and block_table.stride(1) == 1 and pairs.shape[1] == table.shape[1]
    flat = ids.reshape(-1)
    T, Hp = flat.numel(), table.shape[1]
    x = torch.empty((T, Hp), dtype=torch.float32, device=table.device)
    rc = kernels().swb_stream_embed_pairs(flat.data_ptr(), table.data_ptr(), pairs.data_ptr(), 1 if table.dtype == torch.float32 else 0,
                                          table.shape[0], mul_prev, mul_cur, pairs.shape[0] - 1, positions.data_ptr(), slots.data_ptr(),
                                          tokens.data_ptr(), block_table.data_ptr(), block_table.stride(0), tokens.shape[1], ptr(cu_q),
                                          num_seqs, max_q_len, x.data_ptr(), T, Hp, stream_ptr())
    check(rc, "swb_stream_embed_pairs")
    return x
