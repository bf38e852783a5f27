"""Wrappers for the fused LLM glue kernels (norms, RoPE + KV write, gated activations, embedding)."""
from __future__ import annotations

import torch

from .._native import kernels
from .runtime import check, ptr, require_cuda, stream_ptr


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, *, residual: torch.Tensor | None = None,
            out: torch.Tensor | None = None, w_offset: float = 0.0, prefetch: torch.Tensor | None = None,
            prefetch_bytes: int = 0) -> torch.Tensor:
    """out = rmsnorm(x [+ residual]) * (w + w_offset); `residual` (if given) becomes x + residual in place.
    `prefetch`: weights of the kernel that consumes this norm; the first `prefetch_bytes` of them (all when 0) are
    requested into L2 while the norm runs.

    Semantics of the reference rms_norm (candle-llm/src/primitives/nn.rs:21-32): fp32 statistics over the
    last dimension. w_offset = 1 gives the Gemma "+1" convention."""
    require_cuda(x, w)
    x2 = x.reshape(-1, x.shape[-1])
    T, H = x2.shape
    assert x2.stride(1) == 1 and x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16
    if out is None:
        out = torch.empty_like(x2)
    o2 = out.reshape(-1, H)
    r2 = residual.reshape(-1, H) if residual is not None else None
    if prefetch is not None:
        nb = prefetch.numel() * prefetch.element_size()
        nb = min(nb, prefetch_bytes) if prefetch_bytes > 0 else nb
        rc = kernels().swb_rmsnorm_prefetch(x2.data_ptr(), x2.stride(0), ptr(r2), r2.stride(0) if r2 is not None else 0,
                                            w.data_ptr(), o2.data_ptr(), o2.stride(0), T, H, eps, w_offset,
                                            prefetch.data_ptr(), nb, stream_ptr())
    else:
        rc = kernels().swb_rmsnorm(x2.data_ptr(), x2.stride(0), ptr(r2), r2.stride(0) if r2 is not None else 0,
                                   w.data_ptr(), o2.data_ptr(), o2.stride(0), T, H, eps, w_offset, stream_ptr())
    check(rc, "swb_rmsnorm")
    return out.reshape(x.shape)


def layernorm_mod(x: torch.Tensor, *, scale: torch.Tensor | None = None, shift: torch.Tensor | None = None,
                  rows_per_batch: int = 0, gamma: torch.Tensor | None = None, beta: torch.Tensor | None = None,
                  eps: float = 1e-6, out: torch.Tensor | None = None) -> torch.Tensor:
    """out = LN(x) [* gamma + beta] * (1 + scale[b]) + shift[b] (adaLN modulation, one vector per batch)."""
    require_cuda(x)
    x2 = x.reshape(-1, x.shape[-1])
    T, H = x2.shape
    if out is None:
        out = torch.empty_like(x2)
    o2 = out.reshape(-1, H)
    ld_mod = 0
    for m in (scale, shift):
        if m is not None:
            assert m.dtype == torch.bfloat16 and m.stride(-1) == 1
            ld_mod = m.reshape(-1, H).stride(0) if m.numel() > H else H
            if m.dim() >= 2 and m.shape[0] > 1:
                ld_mod = m.stride(0)
    rc = kernels().swb_layernorm_mod(x2.data_ptr(), x2.stride(0), ptr(scale), ptr(shift), ld_mod, rows_per_batch,
                                     ptr(gamma), ptr(beta), o2.data_ptr(), o2.stride(0), T, H, eps, stream_ptr())
    check(rc, "swb_layernorm_mod")
    return out.reshape(x.shape)


def rope_kv_write(qkv: torch.Tensor, positions: torch.Tensor, slot_mapping: torch.Tensor | None,
                  cos: torch.Tensor, sin: torch.Tensor, kcache: torch.Tensor | None, vcache: torch.Tensor | None,
                  n_heads: int, n_kv_heads: int, head_dim: int, *, rot_dim: int | None = None,
                  interleaved: bool = False, q_norm: torch.Tensor | None = None, k_norm: torch.Tensor | None = None,
                  norm_eps: float = 1e-6, norm_w_offset: float = 0.0, block_size: int = 16,
                  v_dim: int | None = None) -> None:
    """In place on qkv [T, (Hq + Hkv) * D + Hkv * v_dim]: per-head q/k RMSNorm (optional), RoPE on q and k; k and v are
    also written to the paged cache [blocks, Hkv, block_size, D | v_dim] at slot_mapping (int64; -1 = skip). bf16, or
    fp32 throughout (projection and caches). v_dim defaults to D."""
    require_cuda(qkv, positions, cos, sin)
    T = qkv.shape[0]
    vd = head_dim if v_dim is None else v_dim
    assert qkv.stride(1) == 1 and positions.dtype == torch.int32 and qkv.dtype in (torch.bfloat16, torch.float32)
    assert qkv.shape[1] >= (n_heads + n_kv_heads) * head_dim + n_kv_heads * vd
    for c in (kcache, vcache):
        assert c is None or c.dtype == qkv.dtype
    assert cos.dtype == torch.float32 and sin.dtype == torch.float32 and cos.is_contiguous() and sin.is_contiguous()
    if slot_mapping is not None:
        assert slot_mapping.dtype == torch.int64
    rd = rot_dim if rot_dim is not None else head_dim
    assert cos.shape[-1] == rd // 2
    rc = kernels().swb_rope_kv_write_ex(qkv.data_ptr(), qkv.stride(0), positions.data_ptr(), ptr(slot_mapping),
                                        cos.data_ptr(), sin.data_ptr(), rd, 1 if interleaved else 0, ptr(q_norm),
                                        ptr(k_norm), norm_eps, norm_w_offset, ptr(kcache), ptr(vcache), block_size, T,
                                        n_heads, n_kv_heads, head_dim, vd, 1 if qkv.dtype == torch.float32 else 0,
                                        stream_ptr())
    check(rc, "swb_rope_kv_write")


def gated_act_mul(gate_up: torch.Tensor, act: str = "silu", out: torch.Tensor | None = None,
                  paired: bool = False, row_gate: torch.Tensor | None = None, limit: float = 0.0) -> torch.Tensor:
    """out[t, f] = act(gate_up[t, f]) * gate_up[t, F + f] (SwiGLU / GeGLU, candle-llm models/llama.rs:1386-1391).
    paired: the projection's rows are interleaved (gate_0, up_0, gate_1, ...), out[t, f] = act(gu[t, 2f]) * gu[t, 2f+1].
    act "clamped": g <- min(g, limit), u <- clamp(u, -limit, limit), out = g sigmoid(1.702 g) (u + 1).
    row_gate fp32 [T] logits (strided): row t is scaled by their sigmoid. bf16 or fp32."""
    require_cuda(gate_up, row_gate)
    g2 = gate_up.reshape(-1, gate_up.shape[-1])
    T, F2 = g2.shape
    F = F2 // 2
    if out is None:
        out = torch.empty((T, F), dtype=gate_up.dtype, device=gate_up.device)
    assert g2.stride(1) == 1 and out.stride(1) == 1 and out.shape == (T, F) and out.dtype == g2.dtype
    assert row_gate is None or (row_gate.dtype == torch.float32 and row_gate.shape == (T,))
    rc = kernels().swb_gated_act_mul_ex(g2.data_ptr(), g2.stride(0), out.data_ptr(), out.stride(0), T, F,
                                        (5 + paired if act == "clamped" else (2 if act in ("gelu", "gelu_tanh") else 1) + 2 * paired), limit, ptr(row_gate),
                                        row_gate.stride(0) if row_gate is not None else 0, 1 if g2.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_gated_act_mul")
    return out.reshape(*gate_up.shape[:-1], F) if gate_up.dim() != 2 else out


def row_rope_kv_write(buf: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, n_heads: int,
                      n_kv_heads: int, head_dim: int, *, v_col: int = 0, rope: tuple[torch.Tensor, torch.Tensor] | None = None,
                      q_norm: torch.Tensor | None = None, k_norm: torch.Tensor | None = None, norm_counts: tuple[int, int] = (0, 0),
                      eps: float = 0.0, v_from_k: bool = False, store_v: bool = False, unit: int = 0) -> None:
    """In place on buf [T, >= (Hq + Hkv) * D]: RMS norms over the whole q and the whole k of a token (fp32 weights q_norm [Hq * D] and
    k_norm [Hkv * D]; norm_counts: how many numbers enter each mean, the rest being zero padding), then rotation of the leading dimensions
    of every head in neighbouring pairs (rope = cos and sin tables fp32 [positions, rot / 2]). k and v go to the paged caches [blocks, Hkv,
    block_size, D | Dv] at `slots` (int64, -1 = skip). Values are the columns from v_col on, or with v_from_k the keys as projected, which
    store_v also copies there. vcache may have heads of its own (their columns then follow one another from v_col on). unit > 0: every q
    and k head is divided by its own root mean square over `unit` columns (the rest being zero padding), without a weight. Without norm
    and rotation the queries are left alone. bf16 or fp32 throughout."""
    require_cuda(buf, positions, slots, kcache, vcache, q_norm, k_norm)
    T, Dv = buf.shape[0], vcache.shape[-1]
    assert buf.stride(1) == 1 and kcache.dtype == vcache.dtype == buf.dtype and kcache.is_contiguous() and vcache.is_contiguous()
    assert kcache.shape[-1] == head_dim and kcache.shape[1] == n_kv_heads and positions.dtype == torch.int32 and slots.dtype == torch.int64
    for w, n in ((q_norm, n_heads), (k_norm, n_kv_heads)):
        assert w is None or (w.dtype == torch.float32 and w.numel() == n * head_dim and w.is_contiguous())
    cos, sin = rope if rope is not None else (None, None)
    rc = kernels().swb_row_rope_kv_write(buf.data_ptr(), buf.stride(0), v_col, n_heads, n_kv_heads, head_dim, Dv,
                                         0 if cos is None else 2 * cos.shape[-1], ptr(q_norm), ptr(k_norm), norm_counts[0], norm_counts[1], eps,
                                         ptr(cos), ptr(sin), positions.data_ptr(), slots.data_ptr(), kcache.data_ptr(), vcache.data_ptr(),
                                         kcache.shape[2], 1 if v_from_k else 0, 1 if store_v else 0, vcache.shape[1], unit, T, 1 if buf.dtype == torch.float32 else 0,
                                         stream_ptr())
    check(rc, "swb_row_rope_kv_write")


def head_mix_weights(talk: torch.Tensor, kv_heads: int) -> torch.Tensor:
    """The mixing matrix [H (to), H (from)] in the layout of `head_mix`: fp32 [H (from), kv_heads, heads per group up to 8s]."""
    H = talk.shape[0]
    per = H // kv_heads
    w = torch.zeros((H, kv_heads, (per + 7) // 8 * 8), dtype=torch.float32, device=talk.device)
    w[:, :, :per] = talk.float().t().reshape(H, kv_heads, per)
    return w


def head_mix(a: torch.Tensor, talk: torch.Tensor, *, gate: torch.Tensor | None = None, out: torch.Tensor | None = None) -> torch.Tensor:
    """Heads that exchange their attention weights. a [T, H, G, Dv]: the weights of each query head applied to the values of all G key/value
    heads (`chunk_attention(all_values=True)`); talk from `head_mix_weights`; gate [T, H] logits (strided rows): head h is scaled by their
    sigmoid. -> [T, H * Dv], out[t, h] = sigmoid(gate[t, h]) sum_g talk[h, g] a[t, g, h // (H / G)]. bf16 or fp32."""
    require_cuda(a, talk, gate, out)
    T, H, G, Dv = a.shape
    assert a.stride()[1:] == (G * Dv, Dv, 1) and talk.shape[:2] == (H, G) and talk.dtype == torch.float32 and talk.is_contiguous()
    assert gate is None or (gate.shape == (T, H) and gate.stride(1) == 1 and gate.dtype == a.dtype)
    if out is None:
        out = torch.empty((T, H * Dv), dtype=a.dtype, device=a.device)
    assert out.shape == (T, H * Dv) and out.stride(1) == 1 and out.dtype == a.dtype
    rc = kernels().swb_head_mix(a.data_ptr(), a.stride(0), talk.data_ptr(), ptr(gate), gate.stride(0) if gate is not None else 0, out.data_ptr(),
                                out.stride(0), T, H, G, Dv, 1 if a.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_head_mix")
    return out


def diff_combine(maps: torch.Tensor, out: torch.Tensor, share: float, eps: float, post: float, width: int | None = None) -> torch.Tensor:
    """Differential attention: out[t, h] = post * N(maps[t, h, 0] - share * maps[t, h, 1]) with N(y) = y / sqrt(mean(y^2) + eps) over the first
    `width` columns. maps [T, H, 2, Dv] (contiguous per token), out [T, H * Dv] strided; bf16 or fp32."""
    require_cuda(maps, out)
    T, H, _, Dv = maps.shape
    assert maps.is_contiguous() and out.shape == (T, H * Dv) and out.stride(1) == 1 and out.dtype == maps.dtype
    rc = kernels().swb_diff_combine(maps.data_ptr(), maps.stride(0), out.data_ptr(), out.stride(0), T, H, Dv, width or Dv, share, eps, post,
                                    1 if maps.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_diff_combine")
    return out


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float, width: int | None = None, out: torch.Tensor | None = None) -> torch.Tensor:
    """out = a N(z) + b N(z^2) + c N(z^3) + e for rows z [T, Fp] (bf16 / fp32), coef fp32 (a, b, c, e), powers element by element
    and N(y) = y / sqrt(mean(y^2) + eps) over the first `width` columns (the rest hold zeros). fp32 statistics."""
    require_cuda(z, coef)
    T, Fp = z.shape
    assert z.stride(1) == 1 and z.dtype in (torch.bfloat16, torch.float32) and coef.dtype == torch.float32 and coef.numel() == 4
    if out is None:
        out = torch.empty((T, Fp), dtype=z.dtype, device=z.device)
    rc = kernels().swb_poly_norm(z.data_ptr(), z.stride(0), out.data_ptr(), out.stride(0), T, width or Fp, Fp, coef.data_ptr(), eps,
                                 1 if z.dtype == torch.float32 else 0, stream_ptr())
    check(rc, "swb_poly_norm")
    return out


def embedding(ids: torch.Tensor, table: torch.Tensor, *, scale: float = 1.0, vocab_start: int = 0,
              out: torch.Tensor | None = None) -> torch.Tensor:
    require_cuda(ids, table)
    assert ids.dtype == torch.int64 and table.is_contiguous()
    flat = ids.reshape(-1)
    T, H = flat.numel(), table.shape[1]
    if out is None:
        out = torch.empty((T, H), dtype=table.dtype, device=table.device)
    rc = kernels().swb_embedding(flat.data_ptr(), table.data_ptr(), out.data_ptr(), T, H, vocab_start,
                                 vocab_start + table.shape[0], scale, stream_ptr())
    check(rc, "swb_embedding")
    return out


def gated_residual(a: torch.Tensor, b: torch.Tensor, gate: torch.Tensor | None = None, rows_per_batch: int = 0,
                   out: torch.Tensor | None = None) -> torch.Tensor:
    """out = a + gate[batch] * b (DiT gated residual) or a + b."""
    require_cuda(a, b)
    H = a.shape[-1]
    a2, b2 = a.reshape(-1, H), b.reshape(-1, H)
    assert a2.is_contiguous() and b2.is_contiguous()
    if out is None:
        out = torch.empty_like(a2)
    ld_gate = 0
    if gate is not None:
        ld_gate = gate.stride(0) if gate.dim() >= 2 and gate.shape[0] > 1 else H
    rc = kernels().swb_gated_residual(a2.data_ptr(), b2.data_ptr(), ptr(gate), ld_gate, rows_per_batch,
                                      out.data_ptr(), a2.shape[0], H, stream_ptr())
    check(rc, "swb_gated_residual")
    return out.reshape(a.shape)


_ARGMAX_SCRATCH: dict[int, torch.Tensor] = {}


def _argmax_scratch(device: torch.device) -> torch.Tensor:
    idx = device.index if device.index is not None else torch.cuda.current_device()
    t = _ARGMAX_SCRATCH.get(idx)
    if t is None:
        t = torch.empty(1 << 20, dtype=torch.uint8, device=device)
        _ARGMAX_SCRATCH[idx] = t
    return t


def argmax(logits: torch.Tensor, allow_mask: torch.Tensor | None = None, out: torch.Tensor | None = None,
           out_vals: torch.Tensor | None = None) -> torch.Tensor:
    """Row-wise argmax (ties -> lowest index) of fp32/bf16 logits; allow_mask: optional uint8 [V]; out_vals:
    optional fp32 [rows] receiving the maxima."""
    require_cuda(logits)
    l2 = logits.reshape(-1, logits.shape[-1])
    assert l2.stride(1) == 1 and l2.dtype in (torch.float32, torch.bfloat16)
    if out is None:
        out = torch.empty(l2.shape[0], dtype=torch.int64, device=logits.device)
    scratch = _argmax_scratch(logits.device)
    rc = kernels().swb_argmax(l2.data_ptr(), 1 if l2.dtype == torch.float32 else 0, l2.stride(0), l2.shape[0],
                              l2.shape[1], ptr(allow_mask), out.data_ptr(), ptr(out_vals), scratch.data_ptr(), scratch.numel(),
                              stream_ptr())
    check(rc, "swb_argmax")
    return out


def sample_device(logits: torch.Tensor, temperature: float, top_k: int, top_p: float, uniforms: torch.Tensor,
                  allow_mask: torch.Tensor | None = None, out: torch.Tensor | None = None,
                  out_prob: torch.Tensor | None = None) -> torch.Tensor:
    """Row-wise draw from softmax(logits / temperature) restricted to the top_k largest weights and the top_p nucleus
    (either limit off with top_k <= 0 / top_p >= 1), on the device. `uniforms`: fp32 [rows] in [0, 1), one per row.
    Returns int64 [rows]; `out_prob` (fp32 [rows]) receives the drawn token's probability within the kept set."""
    require_cuda(logits, uniforms)
    l2 = logits.reshape(-1, logits.shape[-1])
    assert l2.stride(1) == 1 and l2.dtype in (torch.float32, torch.bfloat16) and temperature > 0
    assert uniforms.dtype == torch.float32 and uniforms.numel() == l2.shape[0]
    if out is None:
        out = torch.empty(l2.shape[0], dtype=torch.int64, device=logits.device)
    rc = kernels().swb_sample_device(l2.data_ptr(), 1 if l2.dtype == torch.float32 else 0, l2.stride(0), l2.shape[0], l2.shape[1],
                                     float(temperature), int(top_k), float(top_p), uniforms.data_ptr(), ptr(allow_mask),
                                     out.data_ptr(), ptr(out_prob), stream_ptr())
    check(rc, "swb_sample_device")
    return out


def spec_verify_greedy(target_ids: torch.Tensor, draft: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """target_ids [S, k+1], draft [S, k] (int64) -> (n_accepted int32 [S], next_token int64 [S])."""
    require_cuda(target_ids, draft)
    S, k = draft.shape
    n_acc = torch.empty(S, dtype=torch.int32, device=draft.device)
    nxt = torch.empty(S, dtype=torch.int64, device=draft.device)
    rc = kernels().swb_spec_verify_greedy(target_ids.contiguous().data_ptr(), draft.contiguous().data_ptr(), k, S,
                                          n_acc.data_ptr(), nxt.data_ptr(), stream_ptr())
    check(rc, "swb_spec_verify_greedy")
    return n_acc, nxt
