"""Gunedra decoder on sm_100a kernels: listed layers with a mixer (latent attention or a channel-wise delta rule) and an
optional dense feed-forward, norms on the sublayer outputs only, and an average over depth behind every layer.

Per layer i (x is the fp32 residual stream, N an RMS norm over groups of columns, s1 / s2 per-column scales, m a constant):

    x += m s1 N1(mixer(x))      x += m s2 N2(ff(x))      X_(i+1) = x      x = sum_j dwa_j X_j      (X_0: the embedding rows)

* latent attention: one cached row [c | k_rot] per token serves every head; keys and values are projections of c. A sink joins
  each head's softmax denominator, a sigmoid gate per head scales its output;
* channel delta: q, k, v behind short convolutions, a [dim, vdim] fp32 state per head with a decay per key channel, output norm
  and a low-rank gate;
* feed-forward: down(P(up x)) with P = a N(z) + b N(z^2) + c N(z^3) + e;
* logits: final N, then the embedding table.

How that maps onto the device: s, m and the norm weight are one fp32 vector, so a sublayer's end (norm, join, depth average,
activation copy for the next projection) is one kernel over the row (`ops.stream_norm`). All projections of a mixer's input are
one GEMM. The results X_j stay in a fp32 buffer of the step."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..contracts.errors import Unsupported
from ..engine.kv_pool import LatentGeometry
from ..ops import Branch, DeltaWeights, DepthAverage, LatentWeights, NormWeights
from ..parallel.comm import Communicator
from .config import ChannelDeltaSpec, LatentAttentionSpec, LayerSpec, ModelConfig
from .latent_mixer import LatentDecoder, Ragged
from .llama import StepInputs
from .stack import up8


@dataclass
class _Layer:
    norm1: NormWeights                   # times layer scale and residual multiplier
    dwa: torch.Tensor                    # fp32 [i + 2]
    w_in: torch.Tensor                   # every projection of the mixer's input
    o: torch.Tensor
    latent: LatentWeights | None = None
    rope: tuple[int, float] | None = None
    delta: DeltaWeights | None = None
    low: tuple[tuple[int, torch.Tensor], tuple[int, torch.Tensor]] | None = None   # (column in w_in's output, up projection)
    #                                                                                of the decay and of the gate
    norm2: NormWeights | None = None
    up: torch.Tensor | None = None
    down: torch.Tensor | None = None
    act: torch.Tensor | None = None      # fp32 (a, b, c, e)
    ff: int = 0


class GunedraGpu(LatentDecoder):
    name = "Gunedra"

    def __init__(self, cfg: ModelConfig, comm: Communicator | None = None, device: torch.device | None = None,
                 dtype: torch.dtype = torch.bfloat16):
        super().__init__(cfg, comm, device, dtype)
        self.recurrent = any(isinstance(lay.mixer, ChannelDeltaSpec) for lay in self.stack.layers)
        for i, lay in enumerate(self.stack.layers):
            if isinstance(lay.mixer, ChannelDeltaSpec) and ops.delta_key_width(lay.mixer.dim) is None:
                raise Unsupported(f"layer {i}: key width {lay.mixer.dim} of the delta rule is above 512")
            if isinstance(lay.mixer, LatentAttentionSpec):
                self._check_latent(i, lay.mixer)
        self.layers: list[_Layer] = []

    # ---- cache geometry and scheduling hooks ------------------------------------------------------------------------
    def kv_geometry(self) -> list:
        out = []
        for lay in self.stack.layers:
            m = lay.mixer
            if isinstance(m, LatentAttentionSpec):
                out.append(LatentGeometry(ops.latent_width(self._latent_widths(m)[2], m.rot_dim)))
            else:
                out.append(self._delta_geometry(m))
        return out

    def decode_splits(self, batch: int, max_kv: int) -> tuple[int, ...]:
        return tuple(self._latent_splits(lay.mixer, batch, max_kv) if isinstance(lay.mixer, LatentAttentionSpec) else 1
                     for lay in self.stack.layers)

    def rotations(self) -> set[tuple[int, float]]:
        return {(lay.mixer.rot_dim, lay.mixer.rot_base) for lay in self.stack.layers if isinstance(lay.mixer, LatentAttentionSpec)}

    # ---- weights ------------------------------------------------------------------------------------------------------
    def load_state_dict(self, weights: dict[str, torch.Tensor]) -> "GunedraGpu":
        return self._build(lambda name, *shape: self.tensor(weights, name, *shape))

    def init_random(self, seed: int = 0, std: float = 0.02, low_rank: int | None = None) -> "GunedraGpu":
        """Random weights generated on the device (benchmarks); the low-rank projections get rank `low_rank` (default: the head
        width)."""
        g = torch.Generator(device=self.device).manual_seed(seed)

        def rnd(name: str, *shape: int | None) -> torch.Tensor:
            key = int(name[1:].split(".")[0]) if name[1].isdigit() else 0
            shape = tuple(low_rank or self.stack.layers[key].mixer.dim if s is None else s for s in shape)
            last = name.rsplit(".", 1)[-1]
            if last.startswith("norm") or last.startswith("ls"):
                return torch.ones(shape, device=self.device)
            if last == "dwa":
                t = torch.zeros(shape, device=self.device)
                t[-1] = 1.0
                return t
            return torch.empty(shape, dtype=self.dtype, device=self.device).normal_(0.0, std, generator=g)
        return self._build(rnd)

    def _build(self, get) -> "GunedraGpu":
        W, V, groups = self.width, self.cfg.vocab_size, self.stack.norm_groups
        self.embed = self._mat(get("embed", V, W))
        self.final = NormWeights(self._fp32(get("final.norm", W), self.hp))
        self.layers = []
        for i, spec in enumerate(self.stack.layers):
            L = f"l{i}."

            def scaled(n: int) -> NormWeights:
                w = get(f"{L}norm{n}", W).to(self.device, torch.float32) * get(f"{L}ls{n}", W).to(self.device, torch.float32)
                return NormWeights(self._fp32(w * self.stack.residual_mult, self.hp))
            make = self._latent_layer if isinstance(spec.mixer, LatentAttentionSpec) else self._delta_layer
            lay = make(spec, L + "mix.", get, scaled(1), self._fp32(get(L + "dwa", i + 2)))
            if spec.mlp is not None:
                ff = lay.ff = spec.mlp.ff
                fp = up8(ff)
                lay.norm2 = scaled(2)
                lay.up = torch.zeros((fp, self.hp), dtype=self.dtype, device=self.device)
                lay.up[:ff] = self._mat(get(L + "mlp.up", ff, W))
                lay.down = torch.zeros((self.hp, fp), dtype=self.dtype, device=self.device)
                lay.down[:W, :ff] = get(L + "mlp.down", W, ff).to(self.device, self.dtype)
                lay.act = self._fp32(get(L + "mlp.act", 4))
            self.layers.append(lay)
        return self

    def _latent_layer(self, spec: LayerSpec, p: str, get, norm1: NormWeights, dwa: torch.Tensor) -> _Layer:
        m = spec.mixer
        w_in, latent = self._latent_weights(m, p, get, sink=self._fp32(get(p + "sink", m.heads)))
        return _Layer(norm1, dwa, w_in, self._out(get(p + "o", self.width, m.heads * m.vdim), m.heads, m.vdim, latent.vp), latent=latent,
                      rope=(m.rot_dim, m.rot_base))

    def _delta_layer(self, spec: LayerSpec, p: str, get, norm1: NormWeights, dwa: torch.Tensor) -> _Layer:
        m, W = spec.mixer, self.width
        H, G, D, E, dp, vp = m.heads, m.kv_heads, m.dim, m.vdim, ops.delta_key_width(m.dim), up8(m.vdim)
        hb = up8(H)
        low = {"a1": get(p + "a1", None, W), "g1": get(p + "g1", None, W)}
        ra, rg = low["a1"].shape[0], low["g1"].shape[0]
        rows, conv = self._delta_inputs(m, p, get)
        rows += [self._heads(get(p + "b", H, W), 1, [(H, hb)]), self._heads(low["a1"], 1, [(ra, up8(ra))]),
                 self._heads(low["g1"], 1, [(rg, up8(rg))])]
        col_b = 2 * G * dp + H * vp
        delta = DeltaWeights(H, G, D, dp, E, vp, col_b, conv, self._fp32(get(p + "A_log", H)),
                             self._fp32(get(p + "dt_bias", H * D).reshape(H, D), dp).reshape(-1), self._fp32(get(p + "norm", E), vp))
        a2 = self._heads(get(p + "a2", H * D, ra), H, [(D, dp)], up8(ra))
        g2 = self._heads(get(p + "g2", H * E, rg), H, [(E, vp)], up8(rg))
        return _Layer(norm1, dwa, torch.cat(rows), self._out(get(p + "o", W, H * E), H, E, vp), delta=delta,
                      low=((col_b + hb, a2), (col_b + hb + up8(ra), g2)))

    def weight_bytes(self) -> int:
        ts = [self.embed]
        for lay in self.layers:
            ts += [lay.w_in, lay.o] + ([lay.up, lay.down] if lay.up is not None else [])
            ts += [lay.latent.ukv, lay.latent.uk_t] if lay.latent is not None else [t for _, t in lay.low]
        return sum(t.nbytes for t in ts)

    # ---- forward --------------------------------------------------------------------------------------------------------
    def _latent(self, lay: _Layer, h: torch.Tensor, inp: StepInputs, kv, splits: int, few: Ragged | None,
                many: Ragged | None) -> torch.Tensor:
        w, T = lay.latent, h.shape[0]
        a = torch.empty((T, w.heads, w.vp), dtype=self.dtype, device=self.device)
        self._latent_attend(w, lay.rope, self._linear(h, lay.w_in), inp, kv[0], splits, few, many, a)
        return self._linear(a.view(T, -1), lay.o)

    def _delta(self, lay: _Layer, h: torch.Tensor, inp: StepInputs, kv) -> torch.Tensor:
        proj = self._linear(h, lay.w_in)
        decay, gate = (self._linear(proj[:, c:c + t.shape[1]], t) for c, t in lay.low)
        a = ops.channel_delta(proj, decay, gate, lay.delta, self.cfg.rms_norm_eps, kv[0], kv[1], inp.state_slots, inp.positions,
                              cu_q=inp.cu_q, max_q_len=inp.max_q_len)
        self.launches += 3
        return self._linear(a, lay.o)

    def _ff(self, lay: _Layer, h: torch.Tensor) -> torch.Tensor:
        z = self._linear(h, lay.up)
        self.launches += 1
        return self._linear(ops.poly_norm(z, lay.act, self.cfg.rms_norm_eps, lay.ff, out=z), lay.down)

    def forward_hidden(self, inp: StepInputs, kv: list, *, tap=None) -> torch.Tensor:
        """Runs all layers; kv is `LayeredKvPool.data`. Returns final-normed rows [T | len(logits_rows), Hp]. `tap` (debugging) is
        called with a copy of the residual stream after every layer."""
        if inp.embed_rows is not None or inp.rope_table is not None or inp.deepstack is not None:
            raise Unsupported("Gunedra takes token ids only")
        T, hp, dev, eps = inp.input_ids.numel(), self.hp, self.device, self.cfg.rms_norm_eps
        norm = dict(center=False, groups=self.stack.norm_groups)
        results = torch.empty((len(self.layers) + 1, T, hp), dtype=torch.float32, device=dev)
        x, h = torch.empty((T, hp), dtype=torch.float32, device=dev), torch.empty((T, hp), dtype=self.dtype, device=dev)
        self.launches = 1
        ops.stream_embed(inp.input_ids, self.embed, copies=[h], scale=self.stack.embed_scale, out=results[0])
        few, many = self._split_step(inp)
        splits = inp.attn_splits
        if not isinstance(splits, tuple):
            splits = self.decode_splits(few.n, few.max_kv) if few is not None else (1,) * len(self.layers)
        fuse_final = inp.logits_rows is None
        for i, lay in enumerate(self.layers):
            average, last = DepthAverage(results, i + 1, lay.dwa), i + 1 == len(self.layers)
            end = dict(average=average, norm=self.final if last and fuse_final else None)
            y = self._latent(lay, h, inp, kv[i], splits[i], few, many) if lay.latent is not None else self._delta(lay, h, inp, kv[i])
            first = dict(x_in=results[0]) if i == 0 else {}
            self.launches += 1
            if lay.up is None:
                ops.stream_norm(x, self.width, eps, branch=Branch(y, lay.norm1), out=h, **first, **end, **norm)
            else:
                ops.stream_norm(x, self.width, eps, branch=Branch(y, lay.norm1), out=h, **first, **norm)
                self.launches += 1
                ops.stream_norm(x, self.width, eps, branch=Branch(self._ff(lay, h), lay.norm2), out=h, **end, **norm)
            if tap is not None:
                tap(x[:, :self.width].clone())
        if fuse_final:
            return h
        out = torch.empty((inp.logits_rows.numel(), hp), dtype=self.dtype, device=dev)
        self.launches += 1
        return ops.stream_norm(x, self.width, eps, norm=self.final, out=out, rows=inp.logits_rows, **norm)
