"""Mixture-of-experts pieces: routing plans from a table or from router logits, grouped products (csrc/kernels/moe_routed.cu)."""
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
    weights: torch.Tensor | None = None      # fp32 [T, top] (logits routing)
    ahead: bool = False                      # planned at the start of the step (table routing)

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
                        active[i] if active is not None else None, tiles[i] if tiles is not None else None, ahead=True) for i in range(L)]


_COUNTERS: dict[int, torch.Tensor] = {}


def _counters(device: torch.device) -> torch.Tensor:
    """Per-device counters of the routing kernels, zero between launches."""
    idx = device.index if device.index is not None else torch.cuda.current_device()
    if idx not in _COUNTERS:
        _COUNTERS[idx] = torch.zeros(4096 + 2, dtype=torch.int32, device=device)
    return _COUNTERS[idx]


def logits_routing(logits: torch.Tensor, num_experts: int, top: int, *, rows: torch.Tensor | None = None,
                   renorm: bool = False) -> tuple[RoutingPlan, torch.Tensor | None]:
    """Softmax router: the `top` experts of the largest scores per token, weighted by these scores, as they are or (renorm) divided by
    their sum. logits fp32 [T, >=
    num_experts]. Without `rows` a dense plan; with rows [T, H] a padded plan and the rows copied to their places in the expert-sorted
    buffer."""
    require_cuda(logits, rows)
    assert logits.dtype == torch.float32 and logits.stride(1) == 1 and logits.shape[1] >= num_experts >= top
    T, E, dev, padded = logits.shape[0], num_experts, logits.device, rows is not None
    pairs = T * top
    cap = (pairs + E * (TILE - 1) + TILE - 1) // TILE * TILE if padded else pairs

    def ints(*shape):
        return torch.empty(shape, dtype=torch.int32, device=dev)
    dest, offsets, scratch = ints(T, top), ints(E + 1), ints(2, pairs)
    weights = torch.empty((T, top), dtype=torch.float32, device=dev)
    src, active, tiles = (None, None, ints(cap // TILE)) if padded else (ints(cap), ints(min(E, pairs)), None)
    buf = torch.empty((cap, rows.shape[1]), dtype=rows.dtype, device=dev) if padded else None
    per = 16 // rows.element_size() if padded else 1
    assert not padded or (rows.stride(1) == 1 and rows.stride(0) % per == 0 and rows.shape[1] % per == 0)
    rc = kernels().swb_moe_route(logits.data_ptr(), logits.stride(0), T, E, top, 1 if renorm else 0, TILE if padded else 1, scratch[0].data_ptr(),
                                 scratch[1].data_ptr(), weights.data_ptr(), _counters(dev).data_ptr(), dest.data_ptr(), ptr(src),
                                 offsets.data_ptr(), ptr(active), ptr(tiles), cap, ptr(rows), rows.stride(0) // per if padded else 0, ptr(buf),
                                 rows.shape[1] // per if padded else 0, rows.shape[1] // per if padded else 0, stream_ptr())
    check(rc, "swb_moe_route")
    return RoutingPlan(dest, cap, src, offsets, active, tiles, weights), buf


def gemm_grouped_rows(x: torch.Tensor, w: torch.Tensor, plan: RoutingPlan, *, gather: bool, act: str | None = None,
                      limit: float = 0.0) -> torch.Tensor:
    """out[r] = act(x[src[r] if gather else r] @ w[e]^T) for the rows r of each expert's dense segment; few rows per expert."""
    require_cuda(x, w)
    assert x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.is_contiguous() and x.stride(1) == 1
    E, N, K = w.shape
    assert x.shape[1] == K and not plan.padded
    out = torch.empty((plan.rows, N // 2 if act in ("swiglu_pairs", "geglu_pairs", "clamped_pairs") else N), dtype=torch.bfloat16, device=x.device)
    rc = kernels().swb_gemm_grouped_rows(x.data_ptr(), x.stride(0), plan.src.data_ptr() if gather else None,
                                         plan.offsets.data_ptr(), plan.active.data_ptr(), plan.active.numel(), w.data_ptr(),
                                         out.data_ptr(), out.stride(0), N, K, ACT[act], limit, 1 if plan.ahead else 0, stream_ptr())
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


def routed_gated_ffn(h: torch.Tensor, gate_up: torch.Tensor, down: torch.Tensor, plan: RoutingPlan, act: str, limit: float = 0.0) -> torch.Tensor:
    """Expert outputs [plan.rows, H] in the plan's row order: down_e(act(gate_e x) * (up_e x)), or with act "clamped" the clamped unit of
    `gated_act_mul`. gate_up [E, 2 F, H] with its rows in
    (gate, up) pairs, down [E, H, F]; h as in routed_ffn."""
    from .llm import gated_act_mul

    if h.dtype == torch.float32:
        u = gated_act_mul(gemm_f32(h, gate_up, offsets=plan.offsets, src=plan.src, rows=plan.rows), act, paired=True, limit=limit)
        return gemm_f32(u, down, offsets=plan.offsets, rows=plan.rows)
    if plan.padded:
        return gemm_bf16_grouped(gated_act_mul(gemm_bf16_grouped(h, gate_up, plan.tile_group), act, paired=True, limit=limit), down, plan.tile_group)
    pairs = "clamped_pairs" if act == "clamped" else "geglu_pairs" if act in ("gelu", "gelu_tanh") else "swiglu_pairs"
    return gemm_grouped_rows(gemm_grouped_rows(h, gate_up, plan, gather=True, act=pairs, limit=limit), down, plan, gather=False)
