"""Rotalorn decoder on sm_100a kernels: listed layers whose mixer and feed-forward read one norm and join the stream together.

Per layer (x is the fp32 residual stream, LN a layer norm with bias):

    h = LN(x)      x += mixer(h) + ff(h)

* mixers: grouped attention in a window, its values the projected keys, norms over the whole q and k projections in front of a partial
  rotation; latent attention in a window with low-rank queries and an output gate; differential attention (two capped softmax maps over
  the same values, one subtracted from the other), its queries growing with the position;
* feed-forward: gated dense, or routed experts (softmax scores as they are) plus a shared expert behind a sigmoid gate;
* embedding: token row + a row chosen by the pair (previous token, token); logits: final LN, then the embedding table.

How that maps onto the device: because both sublayers start from h and end in the same sum, their output projections are one GEMM over
[head outputs | feed-forward activations], and one kernel over the row joins it, adds the experts' weighted rows and norms the sum for
the next layer (`ops.stream_norm`). Token ids are paged like keys, so a sequence finds its previous token wherever its pages are. The two
maps of a differential head share a CTA: they are the two query tiles of the prefill kernel and neighbouring query rows of the decode
kernel, so the difference and its norm are part of the attention kernels. Rotations pair i with i + dims / 2 in the checkpoint; the
weights' rows are reordered at load time so that partners are neighbours."""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .. import ops
from ..contracts.errors import Unsupported
from ..engine.kv_pool import KvGeometry, LatentGeometry, TokenGeometry
from ..ops import Branch, Differential, LatentWeights, NormWeights, RoutedRows
from ..parallel.comm import Communicator
from .config import AttentionSpec, DenseSpec, DifferentialSpec, ExpertsSpec, LatentAttentionSpec, ModelConfig
from .latent_mixer import LatentDecoder, Ragged
from .llama import StepInputs, splits_for
from .stack import half_pairs, up8


@dataclass
class _FeedForward:
    """gate_up: rows in (gate, up) pairs. Routed layers: that of the shared expert, with the experts' and the router's weights beside it (the
    router's last used row is the shared expert's gate)."""
    spec: DenseSpec | ExpertsSpec
    gate_up: torch.Tensor                # [2 Fp, Hp]
    router: torch.Tensor | None = None   # [>= E + 1, Hp]
    experts_in: torch.Tensor | None = None      # [E, 2 Fp, Hp]
    experts_out: torch.Tensor | None = None     # [E, Hp, Fp]


@dataclass
class _Layer:
    norm: NormWeights
    w_in: torch.Tensor                   # the mixer's projections of h
    w_out: torch.Tensor                  # [Hp, head output columns + activation columns]
    dk: int                              # padded head widths
    dv: int
    b_in: torch.Tensor | None = None
    q_norm: torch.Tensor | None = None   # fp32 [H * dk]
    k_norm: torch.Tensor | None = None
    rope: tuple | None = None
    latent: LatentWeights | None = None
    share: float = 0.0                   # of the second map
    ff: _FeedForward | None = None


class RotalornGpu(LatentDecoder):
    name = "Rotalorn"

    def __init__(self, cfg: ModelConfig, comm: Communicator | None = None, device: torch.device | None = None,
                 dtype: torch.dtype = torch.bfloat16):
        super().__init__(cfg, comm, device, dtype)
        for i, lay in enumerate(self.stack.layers):
            m = lay.mixer
            if isinstance(m, LatentAttentionSpec):
                self._check_latent(i, m)
            elif max(m.dim, m.vdim) > 1024:
                raise Unsupported(f"layer {i}: attention heads wider than 1024")
        self.layers: list[_Layer] = []
        self.pairs = None
        self._temps: dict[tuple[float, float], torch.Tensor] = {}

    # ---- cache geometry and scheduling hooks ------------------------------------------------------------------------
    def kv_geometry(self) -> list:
        out = []
        for lay in self.stack.layers:
            m = lay.mixer
            if isinstance(m, LatentAttentionSpec):
                out.append(LatentGeometry(ops.latent_width(self._latent_widths(m)[2], m.rot_dim)))
            else:
                out.append(KvGeometry(m.kv_heads, up8(m.dim) * (2 if isinstance(m, DifferentialSpec) else 1), up8(m.vdim)))
        return [*out, TokenGeometry()]

    def decode_splits(self, batch: int, max_kv: int) -> tuple[int, ...]:
        """KV splits per layer: a window (plus the rest of its first tile) is all that a layer reads."""
        def splits(m) -> int:
            if isinstance(m, LatentAttentionSpec):
                return self._latent_splits(m, batch, max_kv)
            window = getattr(m, "window", 0)
            return splits_for(batch, m.kv_heads, min(max_kv, window + 63) if window else max_kv)
        return tuple(splits(lay.mixer) for lay in self.stack.layers)

    @staticmethod
    def _rotation(m: AttentionSpec | LatentAttentionSpec) -> tuple:
        return (m.rot_dim if isinstance(m, LatentAttentionSpec) else m.rot_dims, m.rot_base, m.rot_scaling)

    def rotations(self) -> set[tuple]:
        return {self._rotation(lay.mixer) for lay in self.stack.layers if not isinstance(lay.mixer, DifferentialSpec)}

    def ensure_rope(self, max_positions: int) -> None:
        """Also the query factors of the differential layers by position."""
        if max_positions > self.max_positions:
            pos = torch.arange(1, max_positions + 1, dtype=torch.float64)
            for m in (lay.mixer for lay in self.stack.layers):
                if isinstance(m, DifferentialSpec) and m.temp_coef:
                    t = 1.0 + m.temp_coef * torch.log(torch.floor(pos / m.temp_every) + 1.0)
                    self._temps[(m.temp_coef, m.temp_every)] = t.float().to(self.device)
        super().ensure_rope(max_positions)

    # ---- weights ------------------------------------------------------------------------------------------------------
    def load_state_dict(self, weights: dict[str, torch.Tensor]) -> "RotalornGpu":
        return self._build(lambda name, *shape: self.tensor(weights, name, *shape))

    def init_random(self, seed: int = 0, std: float = 0.02) -> "RotalornGpu":
        """Random weights generated on the device (benchmarks)."""
        g = torch.Generator(device=self.device).manual_seed(seed)

        def rnd(name: str, *shape: int) -> torch.Tensor:
            if name.endswith("norm") or name.endswith("norm1"):
                return torch.ones(shape, device=self.device)
            return torch.empty(shape, dtype=self.dtype, device=self.device).normal_(0.0, std, generator=g)
        return self._build(rnd)

    def _build(self, get) -> "RotalornGpu":
        W, V, b = self.width, self.cfg.vocab_size, self.stack.bigram

        def norm(name: str) -> NormWeights:
            return NormWeights(self._fp32(get(name, W), self.hp), self._fp32(get(name + ".b", W), self.hp))
        self.embed, self.pairs = self._mat(get("embed", V, W)), self._mat(get("bigram", b.buckets + 1, W))
        self.final = norm("final.norm")
        self.layers = []
        for i, spec in enumerate(self.stack.layers):
            m, p = spec.mixer, f"l{i}.mix."
            make = {AttentionSpec: self._attention_layer, LatentAttentionSpec: self._latent_layer, DifferentialSpec: self._differential_layer}
            lay = make[type(m)](m, p, get, norm(f"l{i}.norm1"))
            if spec.mlp is not None:
                lay.ff, down = self._feed_forward(spec.mlp, f"l{i}.mlp.", get)
                lay.w_out = torch.cat([lay.w_out, down], 1)
            self.layers.append(lay)
        return self

    def _attention_layer(self, m: AttentionSpec, p: str, get, norm: NormWeights) -> _Layer:
        W, H, G, D, dp = self.width, m.heads, m.kv_heads, m.dim, up8(m.dim)
        order = torch.tensor(half_pairs(D, m.rot_dims))

        def rows(name: str, n: int) -> torch.Tensor:
            t = get(p + name, n * D, W)
            return self._heads(t.view(n, D, W)[:, order.to(t.device)], n, [(D, dp)])

        def vector(name: str, n: int) -> torch.Tensor:
            t = get(p + name, n * D)
            return self._fp32(t.view(n, D)[:, order.to(t.device)], dp).reshape(-1)
        o = get(p + "o", W, H * D)
        o = o.view(W, H, D)[:, :, order.to(o.device)]       # the values are keys: in their order
        return _Layer(norm, torch.cat([rows("q", H), rows("k", G)]), self._out(o, H, D, dp), dp, dp,
                      b_in=torch.cat([vector("q.b", H), vector("k.b", G)]).to(self.dtype), q_norm=vector("q.norm", H),
                      k_norm=vector("k.norm", G), rope=self._rotation(m))

    def _latent_layer(self, m: LatentAttentionSpec, p: str, get, norm: NormWeights) -> _Layer:
        w_in, latent = self._latent_weights(m, p, get, halves=True)
        return _Layer(norm, w_in, self._out(get(p + "o", self.width, m.heads * m.vdim), m.heads, m.vdim, latent.vp), latent.dn, latent.vp,
                      latent=latent, rope=self._rotation(m))

    def _differential_layer(self, m: DifferentialSpec, p: str, get, norm: NormWeights) -> _Layer:
        W, H, G, D, E, dp, vp = self.width, m.heads, m.kv_heads, m.dim, m.vdim, up8(m.dim), up8(m.vdim)
        w_in = torch.cat([self._heads(get(p + "q", H * 2 * D, W), 2 * H, [(D, dp)]), self._heads(get(p + "k", G * 2 * D, W), 2 * G, [(D, dp)]),
                          self._heads(get(p + "v", G * E, W), G, [(E, vp)])])
        lq1, lk1, lq2, lk2 = (get(p + n, D).double() for n in ("lq1", "lk1", "lq2", "lk2"))
        share = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + m.diff
        return _Layer(norm, w_in, self._out(get(p + "o", W, H * E), H, E, vp), dp, vp, share=share)

    def _feed_forward(self, f: DenseSpec | ExpertsSpec, p: str, get) -> tuple[_FeedForward, torch.Tensor]:
        """(weights, the down projection that shares a GEMM with the mixer's output projection)."""
        W = self.width

        def gated(q: str, ff: int) -> tuple[torch.Tensor, torch.Tensor]:
            return self._pairs(get(q + "gate", ff, W), get(q + "up", ff, W)), self._out(get(q + "down", W, ff), 1, ff, up8(ff))
        if isinstance(f, DenseSpec):
            gate_up, down = gated(p, f.ff)
            return _FeedForward(f, gate_up), down
        E, fp = f.experts, up8(f.ff)
        gate_up, down = gated(p + "shared.", f.shared)
        router = torch.zeros((up8(E + 1), self.hp), dtype=self.dtype, device=self.device)
        router[:E + 1] = torch.cat([self._mat(get(p + "router", E, W)), self._mat(get(p + "shared.sg", 1, W))])
        w = _FeedForward(f, gate_up, router, torch.empty((E, 2 * fp, self.hp), dtype=self.dtype, device=self.device),
                         torch.empty((E, self.hp, fp), dtype=self.dtype, device=self.device))
        for e in range(E):
            w.experts_in[e], w.experts_out[e] = gated(f"{p}e{e}.", f.ff)
        return w, down

    def weight_bytes(self) -> int:
        ts = [self.embed]
        for lay in self.layers:
            ts += [lay.w_in, lay.w_out]
            if lay.latent is not None:
                ts += [lay.latent.ukv, lay.latent.uk_t, lay.latent.uq]
            if lay.ff is not None:
                ts += [t for t in (lay.ff.gate_up, lay.ff.router, lay.ff.experts_in, lay.ff.experts_out) if t is not None]
        return sum(t.nbytes for t in ts)

    # ---- forward --------------------------------------------------------------------------------------------------------
    rows_per_expert_small = 4      # as for the table-routed experts: above it the padded tiles win

    def _attention(self, lay: _Layer, m: AttentionSpec, h: torch.Tensor, inp: StepInputs, kv, splits: int, out: torch.Tensor) -> None:
        T, (kc, vc), nq, nk = h.shape[0], kv, m.heads * lay.dk, m.kv_heads * lay.dk
        fresh = inp.fresh_prefill and inp.cu_q is not None
        buf = torch.empty((T, nq + nk * (2 if fresh else 1)), dtype=self.dtype, device=self.device)
        self._linear(h, lay.w_in, out=buf[:, :nq + nk], bias=lay.b_in)
        ops.row_rope_kv_write(buf, inp.positions, inp.slot_mapping, kc, vc, m.heads, m.kv_heads, lay.dk, v_col=nq + nk,
                              rope=self._rope[lay.rope], q_norm=lay.q_norm, k_norm=lay.k_norm,
                              norm_counts=(m.heads * m.dim, m.kv_heads * m.dim), eps=self.cfg.rms_norm_eps, v_from_k=True, store_v=fresh)
        self.launches += 2
        ops.chunk_attention(buf[:, :nq].view(T, m.heads, lay.dk), kc, vc, inp.block_table, inp.kv_lens, cu_q=inp.cu_q, max_q_len=inp.max_q_len,
                            scale=m.scale, window=m.window, decode=inp.decode, num_splits=splits, out=out,
                            fresh_kv=(buf[:, nq:nq + nk].view(T, m.kv_heads, lay.dk), buf[:, nq + nk:].view(T, m.kv_heads, lay.dv)) if fresh else None)

    def _differential(self, lay: _Layer, m: DifferentialSpec, h: torch.Tensor, inp: StepInputs, kv, splits: int, out: torch.Tensor) -> None:
        T, (kc, vc), nq, nk = h.shape[0], kv, m.heads * 2 * lay.dk, m.kv_heads * 2 * lay.dk
        qkv = self._linear(h, lay.w_in)
        ops.row_rope_kv_write(qkv[:, nq:], inp.positions, inp.slot_mapping, kc, vc, 0, m.kv_heads, 2 * lay.dk, v_col=nk)
        fresh = None
        if inp.fresh_prefill and inp.cu_q is not None:
            fresh = (qkv[:, nq:nq + nk].view(T, m.kv_heads, 2 * lay.dk), qkv[:, nq + nk:].view(T, m.kv_heads, lay.dv))
        self.launches += 2
        diff = Differential(lay.share, 1.0 - m.diff, self.cfg.rms_norm_eps, m.vdim, m.softcap, self._temps.get((m.temp_coef, m.temp_every)))
        ops.chunk_attention(qkv[:, :nq].view(T, m.heads, 2, lay.dk), kc, vc, inp.block_table, inp.kv_lens, cu_q=inp.cu_q,
                            max_q_len=inp.max_q_len, scale=m.scale, decode=inp.decode, num_splits=splits, diff=diff, fresh_kv=fresh, out=out)

    def _activations(self, ff: _FeedForward, h: torch.Tensor, out: torch.Tensor) -> RoutedRows | None:
        """Writes the activations whose down projection shares the output GEMM; returns the routed experts' outputs, if any."""
        T, f, fast = h.shape[0], ff.spec, self.dtype == torch.bfloat16
        if isinstance(f, DenseSpec):
            if fast:
                self.launches += 1 if ops.gated_fused(T, *ff.gate_up.shape) else 2
                ops.linear_gated(h, ff.gate_up, "gelu", out=out)
            else:
                self.launches += 1
                ops.gated_act_mul(self._linear(h, ff.gate_up), "gelu", out=out, paired=True)
            return None
        logits = self._linear(h, ff.router, torch.float32)
        spread = fast and T * f.top > self.rows_per_expert_small * f.experts
        plan, rows = ops.logits_routing(logits, f.experts, f.top, rows=h if spread else None)
        ops.gated_act_mul(self._linear(h, ff.gate_up), "silu", out=out, paired=True, row_gate=logits[:, f.experts])
        y = ops.routed_gated_ffn(rows if spread else h, ff.experts_in, ff.experts_out, plan, "silu")
        self.launches += 4 if T <= 128 and not spread else 6
        return RoutedRows(y, plan.dest, plan.weights)

    def forward_hidden(self, inp: StepInputs, kv: list, *, tap=None) -> torch.Tensor:
        """Runs all layers; kv is `LayeredKvPool.data`. Returns final-normed rows [T | len(logits_rows), Hp]. `tap` (debugging) is
        called with a copy of the residual stream after every layer."""
        if inp.embed_rows is not None or inp.rope_table is not None or inp.deepstack is not None:
            raise Unsupported("Rotalorn takes token ids only")
        T, hp, dev, eps, b = inp.input_ids.numel(), self.hp, self.device, self.cfg.rms_norm_eps, self.stack.bigram
        self.launches = 2
        x = ops.stream_embed_pairs(inp.input_ids, self.embed, self.pairs, b.mul_prev, b.mul_cur, positions=inp.positions,
                                   slots=inp.slot_mapping, tokens=kv[len(self.layers)][0], block_table=inp.block_table, cu_q=inp.cu_q,
                                   num_seqs=inp.num_seqs, max_q_len=inp.max_q_len)
        few, many = (None, None)
        if any(lay.latent is not None for lay in self.layers):
            few, many = self._split_step(inp)
        splits = inp.attn_splits
        if not isinstance(splits, tuple):
            splits = self.decode_splits(few.n, few.max_kv) if few is not None else (1,) * len(self.layers)
        h = ops.stream_norm(x, self.width, eps, norm=self.layers[0].norm, out=torch.empty((T, hp), dtype=self.dtype, device=dev))
        fuse_final = inp.logits_rows is None
        for i, (lay, spec) in enumerate(zip(self.layers, self.stack.layers)):
            m = spec.mixer
            heads = m.heads * lay.dv
            cat = torch.empty((T, lay.w_out.shape[1]), dtype=self.dtype, device=dev)       # [head outputs | activations]
            a = cat[:, :heads]
            routed = self._activations(lay.ff, h, cat[:, heads:]) if lay.ff is not None else None
            if lay.latent is not None:
                self._latent_attend(lay.latent, lay.rope, self._linear(h, lay.w_in), inp, kv[i][0], splits[i], few, many,
                                    a.view(T, m.heads, lay.dv))
            elif isinstance(m, DifferentialSpec):
                self._differential(lay, m, h, inp, kv[i], splits[i], a)
            else:
                self._attention(lay, m, h, inp, kv[i], splits[i], a)
            y = self._linear(cat, lay.w_out)
            last = i + 1 == len(self.layers)
            norm = self.final if last else self.layers[i + 1].norm
            self.launches += 1
            if last and not fuse_final:
                norm = h = None
            else:
                h = torch.empty((T, hp), dtype=self.dtype, device=dev)
            ops.stream_norm(x, self.width, eps, branch=Branch(y, None, extra=routed), norm=norm, out=h)
            if tap is not None:
                tap(x[:, :self.width].clone())
        if fuse_final:
            return h
        out = torch.empty((inp.logits_rows.numel(), hp), dtype=self.dtype, device=dev)
        self.launches += 1
        return ops.stream_norm(x, self.width, eps, norm=self.final, out=out, rows=inp.logits_rows)
