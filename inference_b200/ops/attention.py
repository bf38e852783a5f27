"""Paged and dense attention wrappers (head_dim 128)."""
from __future__ import annotations

import os
from dataclasses import dataclass

import torch

from .._native import kernels
from .runtime import check, ptr, require_cuda, stream_ptr

_DECODE_WS: dict[int, torch.Tensor] = {}


def decode_workspace(device: torch.device, nbytes: int) -> torch.Tensor:
    idx = device.index if device.index is not None else torch.cuda.current_device()
    ws = _DECODE_WS.get(idx)
    if ws is None or ws.numel() < nbytes:
        # zeroed: the head of the buffer holds the split-KV ticket counters, which the kernels leave at zero
        ws = torch.zeros(max(nbytes, 16 << 20), dtype=torch.uint8, device=device)
        _DECODE_WS[idx] = ws
    return ws


def paged_attention(q: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, block_table: torch.Tensor,
                    kv_lens: torch.Tensor, *, cu_q: torch.Tensor | None, max_q_len: int, scale: float,
                    causal: bool = True, decode: bool = False, num_splits: int = 1, softcap: float = 0.0,
                    out: torch.Tensor | None = None, workspace: torch.Tensor | None = None,
                    use_tma: bool = True) -> torch.Tensor:
    """q: [T, Hq, 128] (any token/head strides, unit inner stride); caches [blocks, Hkv, block_size, 128];
    block_table int32 [num_seqs, max_blocks]; kv_lens int32 [num_seqs] (context length including the new
    tokens); cu_q int32 [num_seqs + 1] or None when every sequence has exactly max_q_len query tokens.
    Bottom-right aligned causal mask like the reference SDPA (candle-llm/src/primitives/attention.rs:154-186).
    Prefill (decode=False) with page sizes that divide 128 and no soft cap runs on the tcgen05 kernel, which reads the
    pages through TMA; SWB_PAGED_PREFILL=legacy keeps the mma.sync kernel (comparison runs)."""
    require_cuda(q, kcache, vcache, block_table, kv_lens)
    T, Hq, D = q.shape
    Hkv, bs = kcache.shape[1], kcache.shape[2]
    assert q.stride(2) == 1 and kcache.is_contiguous() and vcache.is_contiguous()
    assert block_table.dtype == torch.int32 and kv_lens.dtype == torch.int32 and block_table.stride(1) == 1
    num_seqs = kv_lens.numel()
    if out is None:
        out = torch.empty((T, Hq * D), dtype=q.dtype, device=q.device)
    if (not decode and D == 128 and softcap == 0.0 and use_tma and bs % 8 == 0 and 128 % bs == 0
            and os.environ.get("SWB_PAGED_PREFILL", "tcgen05") != "legacy"):
        if cu_q is None:
            cu_q = torch.arange(num_seqs + 1, dtype=torch.int32, device=q.device) * max_q_len
        rc = kernels().swb_attn_paged_prefill_tc(q.data_ptr(), q.stride(0), q.stride(1), out.data_ptr(), out.stride(0),
                                                 kcache.data_ptr(), vcache.data_ptr(), block_table.data_ptr(),
                                                 block_table.stride(0), bs, kcache.shape[0], cu_q.data_ptr(),
                                                 kv_lens.data_ptr(), num_seqs, max_q_len, T, Hq, Hkv, scale,
                                                 1 if causal else 0, stream_ptr())
        if rc != -3:
            check(rc, "swb_attn_paged_prefill_tc")
            return out
    ws_ptr, ws_bytes = None, 0
    if decode and num_splits > 1:
        need = kernels().swb_attn_decode_workspace_bytes(num_seqs, Hkv, num_splits)
        if workspace is None:
            workspace = decode_workspace(q.device, need)
        ws_ptr, ws_bytes = workspace.data_ptr(), workspace.numel()
    rc = kernels().swb_attn_paged(q.data_ptr(), q.stride(0), q.stride(1), out.data_ptr(), out.stride(0),
                                  kcache.data_ptr(), vcache.data_ptr(), block_table.data_ptr(), block_table.stride(0),
                                  bs, kcache.shape[0] if use_tma else 0, ptr(cu_q), kv_lens.data_ptr(), num_seqs, max_q_len, Hq, Hkv, D, scale, softcap,
                                  1 if causal else 0, 1 if decode else 0, num_splits, ws_ptr, ws_bytes, stream_ptr())
    check(rc, "swb_attn_paged")
    return out


def dense_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, *, scale: float, causal: bool = False,
                    out: torch.Tensor | None = None) -> torch.Tensor:
    """q [B, Sq, Hq, D], k/v [B, Skv, Hkv, D] (k and v share strides), D = 128 or 64 -> out [B, Sq, Hq*D]. Both widths
    run on the tcgen05 kernel (64-wide heads: one swizzle atom per tile, half the shared memory and MMA work)."""
    require_cuda(q, k, v)
    B, Sq, Hq, D = q.shape
    Skv, Hkv = k.shape[1], k.shape[2]
    assert q.stride(3) == 1 and k.stride(3) == 1 and k.stride() == v.stride()
    assert q.stride(0) == Sq * q.stride(1) and k.stride(0) == Skv * k.stride(1)
    if out is None:
        out = torch.empty((B, Sq, Hq * D), dtype=q.dtype, device=q.device)
    rc = kernels().swb_attn_dense(q.data_ptr(), q.stride(1), q.stride(2), k.data_ptr(), v.data_ptr(), k.stride(1),
                                  k.stride(2), out.data_ptr(), out.stride(1), B, Sq, Skv, Hq, Hkv, D, scale,
                                  1 if causal else 0, stream_ptr())
    check(rc, "swb_attn_dense")
    return out


def narrow_heads_on_kernel() -> bool:
    """Heads narrower than 128 run on the tcgen05 kernel (64 natively, other widths zero-padded to 128) unless
    SWB_NARROW_ATTN=library selects the framework's scaled-dot-product call. SWB_NARROW_ATTN=padded forces the
    zero-padded path for 64-wide heads too (comparison runs)."""
    import os

    return os.environ.get("SWB_NARROW_ATTN", "kernel") != "library"


def dense_attention_padded(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, *, scale: float) -> torch.Tensor:
    """dense_attention for head widths below 128. 64 (SD3 / SDXL blocks) runs natively; other widths (72 in the Qwen3-VL
    tower, 120 in Boogu) are zero-padded to 128 per head, which changes neither q . k nor the first D output columns.
    q [B, Sq, H, D], k / v [B, Skv, Hkv, D] bf16 -> [B, Sq, H * D]."""
    import os

    B, Sq, H, D = q.shape
    if D == 128 or (D == 64 and os.environ.get("SWB_NARROW_ATTN", "kernel") != "padded"):
        return dense_attention(q.contiguous(), k.contiguous(), v.contiguous(), scale=scale)
    assert D < 128
    pad = (0, 128 - D)
    qp, kp, vp = (torch.nn.functional.pad(t, pad).contiguous() for t in (q, k, v))
    out = dense_attention(qp, kp, vp, scale=scale)
    return out.view(B, Sq, H, 128)[..., :D].reshape(B, Sq, H * D)


def set_dense_impl(legacy: bool) -> None:
    """Comparison runs only: True forces the mma.sync kernel for dense attention, False restores the tcgen05 kernel."""
    kernels().swb_attn_dense_set_impl(1 if legacy else 0)


def varlen_causal_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_q: torch.Tensor, max_q_len: int, *,
                            scale: float, out: torch.Tensor | None = None) -> torch.Tensor:
    """Causal self-attention over a packed batch of fresh sequences on the tcgen05 kernel. q [T, Hq, 128], k / v
    [T, Hkv, 128] (views into one QKV buffer are fine), cu_q int32 [num_seqs + 1] -> out [T, Hq * 128]."""
    require_cuda(q, k, v, cu_q)
    T, Hq, D = q.shape
    Hkv = k.shape[1]
    assert D == 128 and q.stride(2) == 1 and k.stride(2) == 1 and k.stride() == v.stride() and cu_q.dtype == torch.int32
    if out is None:
        out = torch.empty((T, Hq * D), dtype=q.dtype, device=q.device)
    rc = kernels().swb_attn_varlen_causal(q.data_ptr(), q.stride(0), q.stride(1), k.data_ptr(), v.data_ptr(), k.stride(0),
                                          k.stride(1), out.data_ptr(), out.stride(0), cu_q.data_ptr(), cu_q.numel() - 1,
                                          max_q_len, T, Hq, Hkv, scale, stream_ptr())
    check(rc, "swb_attn_varlen_causal")
    return out


@dataclass
class Differential:
    """Differential attention: two softmax maps per head over the same values, o = N(a1 - share a2) post, N the RMS norm over the head's
    first `width` value columns. softcap > 0: scores s become softcap tanh(s / softcap). q_temp fp32 [positions]: factor of a query's
    scores in front of the cap."""
    share: float
    post: float
    eps: float
    width: int
    softcap: float = 0.0
    q_temp: torch.Tensor | None = None


def chunk_attention(q: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, block_table: torch.Tensor,
                    kv_lens: torch.Tensor, *, cu_q: torch.Tensor | None, max_q_len: int, scale: float, chunk: int = 0,
                    sink: torch.Tensor | None = None, decode: bool = False, num_splits: int = 1, window: int = 0,
                    fresh_kv: tuple[torch.Tensor, torch.Tensor] | None = None, diff: Differential | None = None,
                    out: torch.Tensor | None = None, kernel: str = "auto", all_values: bool = False,
                    gate: torch.Tensor | None = None) -> torch.Tensor:
    """Causal paged attention with head widths of its own for q / k (D) and v (Dv), optional chunked or windowed masking and sinks.

    q [T, Hq, D] (heads contiguous), caches [blocks, Hkv, block_size, D] and [blocks, Hkv, block_size, Dv], block_table /
    kv_lens / cu_q as in paged_attention -> [T, Hq * Dv]. chunk > 0: position i sees j <= i only when both lie in the same
    run of `chunk` positions, counted from the start of the sequence. window > 0: position i sees only 0 <= i - j < window. sink
    fp32 [Hq]: exp(sink) joins each head's softmax denominator. diff: q [T, Hq, 2, D / 2], the two maps' keys side by side in each
    key row, the result combined. fresh_kv = (k [T, Hkv, D], v [T, Hkv, Dv]) strided views: every sequence starts in this step, so a
    prefill reads its keys there instead of the pages. all_values: the value cache has heads of its own number NV (and fresh values [T, NV,
    Dv]), every query head's weights are applied to all of them -> [T, Hq * NV * Dv]. gate: logits in the shape of the result (strided
    rows), which is scaled by their sigmoid.
    bf16 widths that are multiples of 8 up to 128 run on the tcgen05 kernel (prefill) or the TMA-fed decode kernel; other
    widths, fp32 and non-positive scales on the plain fp32-arithmetic kernel (kernel="simple" forces it)."""
    require_cuda(q, kcache, vcache, block_table, kv_lens, sink, out)
    maps = 1 if diff is None else 2
    T, Hq = q.shape[:2]
    nblk, Hkv, bs, D = kcache.shape
    Dv = vcache.shape[3]
    NV = vcache.shape[1] if all_values else 0
    assert vcache.shape[0] == nblk and vcache.shape[2] == bs and (all_values or vcache.shape[1] == Hkv)
    assert kcache.is_contiguous() and vcache.is_contiguous() and not (diff is not None and (all_values or gate is not None))
    problems = Hkv * max(NV, 1)          # of a sequence in decoding
    assert q.shape[2:] == ((D,) if diff is None else (2, D // 2)) and q.stride(-1) == 1 and q.stride(1) == D
    assert q.dtype == kcache.dtype == vcache.dtype and (diff is None or (D % 2 == 0 and q.stride(2) == D // 2))
    assert block_table.dtype == torch.int32 and kv_lens.dtype == torch.int32 and block_table.stride(1) == 1
    assert sink is None or (sink.dtype == torch.float32 and sink.numel() == Hq and sink.is_contiguous())
    temp = diff.q_temp if diff is not None else None
    assert temp is None or (temp.is_cuda and temp.dtype == torch.float32 and temp.is_contiguous())
    num_seqs = kv_lens.numel()
    if out is None:
        out = torch.empty((T, Hq * max(NV, 1) * Dv), dtype=q.dtype, device=q.device)
    assert out.shape == (T, Hq * max(NV, 1) * Dv) and out.stride(1) == 1 and out.dtype == q.dtype
    assert gate is None or (gate.shape == out.shape and gate.stride(1) == 1 and gate.dtype == q.dtype)
    gate_args = (NV, ptr(gate), gate.stride(0) if gate is not None else 0)
    if q.dtype == torch.bfloat16 and kernel == "auto" and scale > 0 and max(D, Dv) <= 128 and D % (8 * maps) == 0 and Dv % 8 == 0:
        decode = decode and max_q_len * maps * (Hq // Hkv) <= 16 and bs == 16
        ws_ptr, ws_bytes, k, v, ks, vs, table = None, 0, kcache, vcache, 0, 0, block_table
        if decode and num_splits > 1:
            ws = decode_workspace(q.device, kernels().swb_attn_decode_workspace_bytes(num_seqs, problems, num_splits))
            ws_ptr, ws_bytes = ws.data_ptr(), ws.numel()
        if not decode:
            if cu_q is None:
                cu_q = torch.arange(num_seqs + 1, dtype=torch.int32, device=q.device) * max_q_len
            if fresh_kv is not None:
                k, v = fresh_kv
                assert k.stride(2) == 1 and v.stride(2) == 1 and k.stride(1) == D and v.stride(1) == Dv
                ks, vs, table = k.stride(0), v.stride(0), None
        d = diff or Differential(0.0, 1.0, 0.0, Dv)
        rc = kernels().swb_attn_ext(q.data_ptr(), q.stride(0), k.data_ptr(), ks, v.data_ptr(), vs, out.data_ptr(),
                                    out.stride(0), ptr(table), block_table.stride(0), bs, nblk, ptr(cu_q),
                                    kv_lens.data_ptr(), num_seqs, max_q_len, T, Hq, Hkv, D, Dv, scale, chunk, ptr(sink),
                                    1 if decode else 0, num_splits, ws_ptr, ws_bytes, window, 0 if diff is None else 1, d.share, d.eps, d.post,
                                    d.softcap, ptr(temp), d.width, *gate_args, stream_ptr())
        if rc != -3:
            check(rc, "swb_attn_ext")
            return out
    res = out if diff is None else torch.empty((T, Hq, 2, Dv), dtype=q.dtype, device=q.device)
    rc = kernels().swb_attn_simple(q.data_ptr(), q.stride(0), kcache.data_ptr(), vcache.data_ptr(), res.data_ptr(),
                                   res.stride(0), block_table.data_ptr(), block_table.stride(0), bs, ptr(cu_q),
                                   kv_lens.data_ptr(), num_seqs, max_q_len, T, Hq * maps, Hkv, D // maps, Dv, 0, scale, chunk, ptr(sink),
                                   window, diff.softcap if diff is not None else 0.0, ptr(temp), maps, *gate_args,
                                   1 if q.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_attn_simple")
    if diff is not None:
        from .llm import diff_combine

        diff_combine(res, out, diff.share, diff.eps, diff.post, diff.width)
    return out


def exchange_decode_fits(heads: int, kv_heads: int, dim: int, value_heads: int, v_dim: int, q_len: int = 1) -> bool:
    """Whether decoding with exchanged weights runs on the kernel that takes all heads of a sequence in one CTA (the limits of
    csrc/kernels/attention_exchange.cu): rows and value columns within its accumulators, two pages in shared memory."""
    rows, cols = heads * q_len, value_heads * v_dim
    page = 2048 * ((dim + 63) // 64 * kv_heads + (v_dim + 63) // 64 * value_heads)
    fixed = (rows * ((dim + 15) // 16 * 32 + 16) + 15) // 16 * 16 + 2 * 64 * 52 + 1280
    return (rows <= 64 and max(dim, v_dim) <= 128 and dim % 8 == 0 and v_dim % 8 == 0 and max(kv_heads, value_heads) <= 16
            and cols <= (1024 if rows <= 16 else 512 if rows <= 32 else 256) and fixed + 2 * page <= 227 * 1024)


def exchange_attention(q: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, block_table: torch.Tensor, kv_lens: torch.Tensor, *,
                       cu_q: torch.Tensor | None, max_q_len: int, scale: float, talk: torch.Tensor, sink: torch.Tensor | None = None,
                       gate: torch.Tensor | None = None, window: int = 0, decode: bool = False, num_splits: int = 1,
                       fresh_kv: tuple[torch.Tensor, torch.Tensor] | None = None, kernel: str = "auto") -> torch.Tensor:
    """Attention whose heads exchange their weights: head h applies sum_g talk[h, g] (weights of head g) to the values of its own key/value
    head and is scaled by the sigmoid of gate [T, Hq] logits. talk from `head_mix_weights`; vcache [blocks, NV, block_size, Dv] with NV Dv = Hkv
    times the value width; the rest as in `chunk_attention` -> [T, Hq * width]. bf16 decode steps run on one kernel over all heads and a merge
    that mixes and gates (`exchange_decode_fits`), everything else on chunk_attention over all values and `head_mix`."""
    from .llm import head_mix

    T, H, D = q.shape
    nblk, G, bs, _ = kcache.shape
    NV, Dv = vcache.shape[1], vcache.shape[3]
    vp = NV * Dv // G
    if (decode and cu_q is None and q.dtype == torch.bfloat16 and kernel == "auto" and bs == 16 and scale > 0
            and exchange_decode_fits(H, G, D, NV, Dv, max_q_len)):
        require_cuda(q, kcache, vcache, block_table, kv_lens, talk, sink, gate)
        S = kv_lens.numel()
        assert T == S * max_q_len and q.stride(2) == 1 and q.stride(1) == D and kcache.is_contiguous() and vcache.is_contiguous()
        assert vcache.shape[0] == nblk and kcache.dtype == vcache.dtype == q.dtype and block_table.dtype == kv_lens.dtype == torch.int32
        assert talk.shape[:2] == (H, G) and talk.dtype == torch.float32 and talk.is_contiguous() and block_table.stride(1) == 1
        assert sink is None or (sink.dtype == torch.float32 and sink.numel() == H)
        assert gate is None or (gate.shape == (T, H) and gate.stride(1) == 1 and gate.dtype == q.dtype)
        n = max(1, min(32, num_splits))
        ws = torch.empty(kernels().swb_exchange_workspace_bytes(S, H, max_q_len, NV * Dv, n), dtype=torch.uint8, device=q.device)
        out = torch.empty((T, H * vp), dtype=q.dtype, device=q.device)
        rc = kernels().swb_exchange_decode(q.data_ptr(), q.stride(0), kcache.data_ptr(), vcache.data_ptr(), out.data_ptr(), out.stride(0),
                                           block_table.data_ptr(), block_table.stride(0), nblk, kv_lens.data_ptr(), S, max_q_len, H, G, D, NV, Dv,
                                           vp, scale, window, ptr(sink), talk.data_ptr(), ptr(gate), gate.stride(0) if gate is not None else 0, n,
                                           ws.data_ptr(), ws.numel(), stream_ptr())
        check(rc, "swb_exchange_decode")
        return out
    a = chunk_attention(q, kcache, vcache, block_table, kv_lens, cu_q=cu_q, max_q_len=max_q_len, scale=scale, window=window, sink=sink,
                        decode=decode, num_splits=num_splits, fresh_kv=fresh_kv, kernel=kernel, all_values=True)
    return head_mix(a.view(T, H, G, vp), talk, gate=gate)
