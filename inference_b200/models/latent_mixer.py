"""Latent attention layers of the decoders whose config lists its layers: padded weights, KV splits, how a step is divided between
attention in the latent space and attention on expanded keys, and the layer itself up to the output projection."""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from .. import ops
from ..contracts.errors import Unsupported
from ..ops import LatentWeights, QueryRotation
from .config import LatentAttentionSpec
from .llama import StepInputs
from .stack import StackDecoder, half_pairs, up8


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass
class Ragged:
    """Sequences of a step that take one attention path. `rows` int32: their tokens, or None when they are all of the step."""
    n: int
    tokens: int
    max_q: int
    max_kv: int
    seqs: torch.Tensor | None = None
    rows: torch.Tensor | None = None
    cu: torch.Tensor | None = None       # token offsets among `rows` (latent space) or in the step
    spans: list[tuple[int, int]] = field(default_factory=list)    # expanded path with earlier context: (new tokens, context length)
    q_row: torch.Tensor | None = None    # int32 [T]: index in `rows` of each token, -1: not one of them
    _keys: dict[int, tuple] = field(default_factory=dict)

    def keys(self, window: int, device: torch.device) -> tuple[torch.Tensor, torch.Tensor | None, int]:
        """(offsets of the key rows, first key row of each sequence or None, number of key rows) for layers with this window."""
        if window not in self._keys:
            first = [max(0, n - q - window + 1) if window else 0 for q, n in self.spans]
            ends = [0]
            for (_, n), f in zip(self.spans, first):
                ends.append(ends[-1] + n - f)
            both = torch.tensor(ends + first, dtype=torch.int32).to(device, non_blocking=True)
            self._keys[window] = (both[:len(ends)], both[len(ends):] if any(first) else None, ends[-1])
        return self._keys[window]


class LatentDecoder(StackDecoder):
    few_tokens = 16      # measured on B200: up to so many tokens of a sequence attend in the latent space

    @staticmethod
    def _latent_widths(m: LatentAttentionSpec) -> tuple[int, int, int, int]:
        """Padded dim, rot_dim, kv_rank, vdim."""
        return _up(m.dim, 16), up8(m.rot_dim), _up(m.kv_rank, 64), _up(m.vdim, 16)

    def _check_latent(self, i: int, m: LatentAttentionSpec) -> None:
        if ops.latent_width(self._latent_widths(m)[2], m.rot_dim) > 1024:
            raise Unsupported(f"layer {i}: a cached row of {m.kv_rank} + {m.rot_dim} is above 1024")

    @staticmethod
    def _latent_splits(m: LatentAttentionSpec, batch: int, max_kv: int) -> int:
        """KV splits: about one CTA per SM, no split below two 64-key tiles; a window bounds the keys (with the rest of its tiles)."""
        keys = min(max_kv, m.window + 63) if m.window else max_kv
        want, s = min(148 // (batch * ((m.heads + 31) // 32)), (keys + 127) // 128, 32), 1
        while s * 2 <= want:
            s *= 2
        return s

    def _latent_weights(self, m: LatentAttentionSpec, p: str, get, *, sink: torch.Tensor | None = None,
                        halves: bool = False) -> tuple[torch.Tensor, LatentWeights]:
        """(all projections of the layer's input, the rest). halves: the checkpoint's rotation pairs are (i, i + rot_dim / 2)."""
        W, H, R, Q = self.width, m.heads, m.kv_rank, m.q_rank
        dn, rp, rk, vp = self._latent_widths(m)
        order = torch.tensor(half_pairs(m.rot_dim, m.rot_dim) if halves else list(range(m.rot_dim)))

        def turn(t: torch.Tensor, heads: int, front: int) -> torch.Tensor:       # the rotated rows behind the first `front` of every head
            t = t.reshape(heads, front + m.rot_dim, -1)
            return torch.cat([t[:, :front], t[:, front:][:, order.to(t.device)]], 1).reshape(-1, t.shape[2])
        q = turn(get(p + ("uq" if Q else "q"), H * (m.dim + m.rot_dim), Q or W), H, m.dim)
        qk = _up(Q, 16)
        q = self._heads(q, H, [(m.dim, dn), (m.rot_dim, rp)], qk if Q else None)
        w_in = torch.cat([self._heads(get(p + "dq", Q, W), 1, [(Q, qk)]) if Q else q,
                          self._heads(turn(get(p + "dkv", R + m.rot_dim, W), 1, R), 1, [(R, rk), (m.rot_dim, rp)]),
                          self._heads(get(p + "g", H, W), 1, [(H, up8(H))])])
        uk = self._heads(get(p + "uk", H * m.dim, R), H, [(m.dim, dn)], rk).view(H, dn, rk)
        uv = self._heads(get(p + "uv", H * m.vdim, R), H, [(m.vdim, vp)], rk).view(H, vp, rk)
        low = dict(q_rank=Q, qk=qk, q_norm=self._fp32(get(p + "dq.norm", Q), qk), uq=q) if Q else {}
        return w_in, LatentWeights(H, m.dim, dn, m.rot_dim, rp, R, rk, m.vdim, vp, m.scale, self._fp32(get(p + "dkv.norm", R), rk), sink,
                                   torch.cat([uk.view(H * dn, rk), uv.view(H * vp, rk)]), uk.transpose(1, 2).contiguous(),
                                   window=m.window, **low)

    def _split_step(self, inp: StepInputs) -> tuple[Ragged | None, Ragged | None]:
        """(few, many): sequences with few new tokens attend in the latent space, where all heads share the cached rows; for the
        others expanding the latents into keys and values of every head costs less than it saves. A decode step, and 32-bit
        mode, is all few."""
        T, S = inp.input_ids.numel(), inp.num_seqs
        spans = inp.spans
        if spans is None:
            return Ragged(S, T, inp.max_q_len, 0, cu=inp.cu_q), None
        limit = self.few_tokens if self.dtype == torch.bfloat16 else max(q for q, _ in spans)
        few, many = [i for i in range(S) if spans[i][0] <= limit], [i for i in range(S) if spans[i][0] > limit]
        dev_i32 = lambda v: torch.tensor(v, dtype=torch.int32).to(self.device, non_blocking=True)   # noqa: E731
        starts = [0]
        for q, _ in spans:
            starts.append(starts[-1] + q)

        def ragged(ids: list[int], is_many: bool) -> Ragged | None:
            if not ids:
                return None
            r = Ragged(len(ids), sum(spans[i][0] for i in ids), max(spans[i][0] for i in ids), max(spans[i][1] for i in ids))
            if len(ids) < S:
                r.seqs = dev_i32(ids)
            if is_many:
                if len(ids) < S or any(q != n for q, n in spans):       # earlier context: keys come from the cache
                    r.spans = [spans[i] for i in ids]
            elif len(ids) < S:
                rows = [t for i in ids for t in range(starts[i], starts[i + 1])]
                q_row, ends = [-1] * T, [0]
                for k, t in enumerate(rows):
                    q_row[t] = k
                for i in ids:
                    ends.append(ends[-1] + spans[i][0])
                r.rows, r.q_row, r.cu = dev_i32(rows), dev_i32(q_row), dev_i32(ends)
            else:
                r.cu = inp.cu_q
            return r
        return ragged(few, False), ragged(many, True)

    def _latent_attend(self, w: LatentWeights, rope: tuple, proj: torch.Tensor, inp: StepInputs, cache: torch.Tensor, splits: int,
                       few: Ragged | None, many: Ragged | None, out: torch.Tensor) -> None:
        """From the projections of the layer's input to the gated head outputs out [T, heads, vp] (strided)."""
        T, dev = proj.shape[0], self.device
        cos, sin = self._rope[rope]
        table, lens, fast = inp.block_table, inp.kv_lens, self.dtype == torch.bfloat16
        cu_q = inp.cu_q
        if many is not None and not ops.latent_prefill_supported(w):
            # heads wider than the prefill kernel: everything attends in the latent space
            few, many = Ragged(inp.num_seqs, T, inp.max_q_len, max(n for _, n in inp.spans), cu=cu_q), None
        q_abs = torch.empty((few.tokens, w.heads, w.width), dtype=self.dtype, device=dev) if few is not None else None
        q_row = few.q_row if few is not None else None
        turn = None
        self.launches += 1
        if w.q_rank:
            ops.latent_prep(proj, w, self.cfg.rms_norm_eps, cos, sin, inp.positions, inp.slot_mapping, cache)
            queries = self._linear(proj[:, :w.qk], w.uq)
            if many is None and fast:
                turn = QueryRotation(cos, sin, inp.positions, w.dn, w.rot, w.rp, w.rc)      # with the key projection below
            else:
                self.launches += 1
                ops.rotate_queries(queries, w, cos, sin, inp.positions, q_abs, q_row)
        else:
            ops.latent_prep(proj, w, self.cfg.rms_norm_eps, cos, sin, inp.positions, inp.slot_mapping, cache, q_abs, q_row)
            queries = proj[:, :w.col_c]
        gate = proj[:, w.col_gate:w.col_gate + w.heads]
        if many is not None:
            if cu_q is None:
                cu_q = torch.arange(inp.num_seqs + 1, dtype=torch.int32, device=dev) * inp.max_q_len
            rows, cu_k = proj[:, w.col_c:w.col_gate], None
            if many.spans:
                cu_k, first, n_keys = many.keys(w.window, dev)
                rows = ops.latent_gather(cache, table, cu_k, n_keys, many.seqs, first)
                self.launches += 1
            expanded = self._linear(rows[:, :w.rk], w.ukv)
            ops.latent_prefill(queries, expanded, rows[:, w.rk:w.rk + w.rp], w, out.view(T, -1), cu_q=cu_q, max_q_len=many.max_q, gate=gate,
                               seqs=many.seqs, cu_k=cu_k)
            self.launches += 1
        if few is not None:
            q = queries.view(T, w.heads, w.dn + w.rp)[..., :w.dn]
            ops.head_product(q, w.uk_t, q_abs[..., :w.rk], rows_in=few.rows, rows_out=None, rotate=turn)
            if few.seqs is not None:
                table, lens = table[few.seqs], lens[few.seqs]
            ragged = dict(cu_q=few.cu, max_q_len=few.max_q)
            if fast and ops.latent_decode_supported(w, cache.shape[1]):
                lat = ops.latent_decode(q_abs, cache, table, lens, w, num_splits=splits, **ragged)
            else:
                lat = ops.latent_attention_simple(q_abs, cache, table, lens, w, **ragged)
            ops.head_product(lat, w.uv, out, gate=gate, sink=w.sink, rows_out=few.rows)
            self.launches += 3
