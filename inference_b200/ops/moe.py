"""Mixture-of-experts pieces whose routing is known before the layer runs (csrc/kernels/moe_routed.cu)."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .._native import kernels
from .gemm import ACT, gemm_bf16_grouped, gemm_f32
from .runtime import check, ptr, require_cuda, stream_ptr

TILE = 128      # row tile of the tcgen05 grouped GEMM


@dataclass
class RoutingPlan:
    """Where a layer's (token, slot) pairs live in its expert-sorted buffer. dest int32 [T, top]: buffer row of each pair.
    Padded plans (prefill) name the expert of every 128-row tile; dense plans (few rows per expert) carry the segment
    offsets, the source token of every row and the list of experts that got tokens."""
    dest: torch.Tensor
    rows: int
    src: torch.Tensor | None = None
    offsets: torch.Tensor | None = None
    active: torch.Tensor | None = None
    tile_group: torch.Tensor | None = None

    @property
    def padded(self) -> bool:
        return self.tile_group is not None


def table_routing(ids: torch.Tensor, tables: torch.Tensor, num_experts: int, *, padded: bool) -> list[RoutingPlan]:
    """Plans for all layers of one step in one launch. ids int64 [T]; tables int32 [layers, vocab, top] name the experts of
    every token id (the router of the layer: no logits, equal weights)."""
    require_cuda(ids, tables)
    assert ids.dtype == torch.int64 and tables.dtype == torch.int32 and tables.is_contiguous()
    L, V, top = tables.shape
    T, E, dev = ids.numel(), num_experts, ids.device
    pairs = T * top
    rows = (pairs + E * (TILE - 1) + TILE - 1) // TILE * TILE if padded else pairs

    def ints(*shape):
        return torch.empty(shape, dtype=torch.int32, device=dev)
    dest, offsets = ints(L, T, top), ints(L, E + 1)
    src = None if padded else ints(L, rows)
    active = None if padded else ints(L, min(E, pairs))
    tiles = ints(L, rows // TILE) if padded else None
    rc = kernels().swb_moe_table_plan(ids.data_ptr(), T, tables.data_ptr(), L, V, top, E, TILE if padded else 1,
                                      dest.data_ptr(), ptr(src), offsets.data_ptr(), ptr(active), ptr(tiles), rows,
                                      stream_ptr())
    check(rc, "swb_moe_table_plan")
    return [RoutingPlan(dest[i], rows, src[i] if src is not None else None, offsets[i],
                        active[i] if active is not None else None, tiles[i] if tiles is not None else None) for i in range(L)]


def gemm_grouped_rows(x: torch.Tensor, w: torch.Tensor, plan: RoutingPlan, *, gather: bool, act: str | None = None) -> torch.Tensor:
    """out[r] = act(x[src[r] if gather else r] @ w[e]^T) for the rows r of each expert's dense segment; few rows per expert."""
    require_cuda(x, w)
    assert x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.is_contiguous() and x.stride(1) == 1
    E, N, K = w.shape
    assert x.shape[1] == K and not plan.padded
    out = torch.empty((plan.rows, N), dtype=torch.bfloat16, device=x.device)
    rc = kernels().swb_gemm_grouped_rows(x.data_ptr(), x.stride(0), plan.src.data_ptr() if gather else None,
                                         plan.offsets.data_ptr(), plan.active.data_ptr(), plan.active.numel(), w.data_ptr(),
                                         out.data_ptr(), out.stride(0), N, K, ACT[act], stream_ptr())
    check(rc, "swb_gemm_grouped_rows")
    return out


def routed_ffn(h: torch.Tensor, up: torch.Tensor, down: torch.Tensor, plan: RoutingPlan, act: str) -> torch.Tensor:
    """Expert outputs [plan.rows, H] in the plan's row order: down_e(act(up_e x)), ungated. h is the expert-sorted buffer of a
    padded plan (every token's row stored at its dest rows), or the plain [T, H] rows of a dense plan."""
    if h.dtype == torch.float32:
        u = gemm_f32(h, up, act=act, offsets=plan.offsets, src=plan.src, rows=plan.rows)
        return gemm_f32(u, down, offsets=plan.offsets, rows=plan.rows)
    if plan.padded:
        return gemm_bf16_grouped(gemm_bf16_grouped(h, up, plan.tile_group, act=act), down, plan.tile_group)
    return gemm_grouped_rows(gemm_grouped_rows(h, up, plan, gather=True, act=act), down, plan, gather=False)
