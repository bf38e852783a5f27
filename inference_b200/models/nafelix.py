"""Nafelix decoder on sm_100a kernels: listed layers over several residual streams, a range of them run several times in a row.

Per sublayer (x_1 .. x_S the fp32 streams, all equal to the embedding row at the start, N an RMS norm, conv a short causal convolution over
time on every channel):

    h = N(sum_s read[s] x_s) w      y = sublayer(h + conv(h))      x_t <- sum_s mix[s, t] x_s + put[t] y

* mixer "parallel": attention in a window whose heads exchange their weights, with sinks and a gate per head, beside a delta rule with
  short convolutions and one decay per head; each result is normed over the width and the two are averaged;
* mixer "attention": attention in a window with sinks and projection biases, queries and keys of unit root mean square per head, a gate
  per output element;
* feed-forward: dense with xIELU, or routed experts with clamped gated units, their softmax scores divided by the sum of the chosen ones;
* loop: every pass has its own cache and states; logits: N of the sum of the streams, then a table of their own.

How that maps onto the device: everything between two sublayers is one kernel over a token (`ops.hyper_step`): the norms of a parallel
mixer's two results, the weighted expert rows, the join of all streams, what the next sublayer reads, its norm and, when every sequence
brings one token, its convolution, whose window is part of a sequence's state slot; prompts run the convolution as one more kernel. All
projections of a mixer's input are one GEMM. Exchanged weights are never formed: a head's mixed weights applied to its values equal
sum_g talk[h, g] (weights of head g applied to the values of h's group), so the attention kernels apply every head's weights to all value
heads (cached side by side, up to 128 columns to a tile) and their results are mixed and gated behind it (`ops.exchange_attention`). Rotations pair i with i + dims / 2 in the
checkpoint; the weights' rows are reordered at load time so that partners are neighbours; the unit norms stand in front of the rotation,
which does not change a head's length."""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .. import ops
from ..contracts.errors import Unsupported
from ..engine.kv_pool import KvGeometry, WindowGeometry
from ..ops import DeltaWeights, HyperBranch, NormWeights, RoutedRows, ShortConv, StreamMix
from ..ops.hyper import MAX_STREAMS, MAX_WIDTH
from ..parallel.comm import Communicator
from .config import AttentionSpec, DenseSpec, ExpertsSpec, HeadDeltaSpec, ModelConfig, ParallelSpec
from .llama import StepInputs, splits_for
from .stack import StackDecoder, half_pairs, up8


@dataclass
class _Sublayer:
    """What stands in front of and behind a mixer or a feed-forward."""
    norm: NormWeights
    read: torch.Tensor                   # fp32 [S]
    join: StreamMix
    conv: torch.Tensor                   # fp32 [taps, Hp]


@dataclass
class _Attention:
    """dk, dv: padded widths of q / k and of a cached value head; value_heads of them (exchanged weights: several heads' values in one)."""
    spec: AttentionSpec
    dk: int
    dv: int
    value_heads: int
    sink: torch.Tensor
    o: torch.Tensor
    rope: tuple[int, float] | None
    talk: torch.Tensor | None = None     # exchanged weights: `ops.head_mix_weights`
    unit: int = 0                        # unit norms of q and k: their real width

    @property
    def cols(self) -> tuple[int, int, int]:
        """Columns of q, k, v in the projections."""
        m = self.spec
        return m.heads * self.dk, m.kv_heads * self.dk, self.value_heads * self.dv


@dataclass
class _Delta:
    weights: DeltaWeights
    o: torch.Tensor
    col: int                             # first column in the projections
    col_gate: int                        # of the output gate, counted from there


@dataclass
class _FeedForward:
    """Dense: up, down and the activation's parameters. Routed: up = the experts' rows in (gate, up) pairs [E, 2 Fp, Hp], down [E, Hp, Fp]."""
    spec: DenseSpec | ExpertsSpec
    up: torch.Tensor
    down: torch.Tensor
    act: tuple[float, float] = (0.0, 0.0)
    router: torch.Tensor | None = None


@dataclass
class _Layer:
    w_in: torch.Tensor                   # every projection of the mixer's input
    attention: _Attention
    mixer: _Sublayer
    b_in: torch.Tensor | None = None
    delta: _Delta | None = None          # parallel mixers
    norms: tuple[NormWeights, NormWeights] | None = None      # of their two results, times one half
    ff: _FeedForward | None = None
    ffn: _Sublayer | None = None


def values_together(kv_heads: int, width: int, limit: int = 128) -> int:
    """How many heads' values of `width` columns share a cached value head of at most `limit` columns (a divisor of kv_heads)."""
    return max(n for n in range(1, kv_heads + 1) if kv_heads % n == 0 and (n == 1 or n * width <= limit))


class NafelixGpu(StackDecoder):
    name = "Nafelix"
    recurrent = True

    def __init__(self, cfg: ModelConfig, comm: Communicator | None = None, device: torch.device | None = None,
                 dtype: torch.dtype = torch.bfloat16):
        super().__init__(cfg, comm, device, dtype)
        self.runs = [i for i, _ in self.stack.runs()]
        self.streams, self.taps = self.stack.streams, self.stack.canon_taps
        if self.streams > MAX_STREAMS or self.hp > MAX_WIDTH:
            raise Unsupported(f"{self.streams} streams of {self.width} columns: at most {MAX_STREAMS} of {MAX_WIDTH}")
        for i, lay in enumerate(self.stack.layers):
            m = lay.mixer
            a = m.left if isinstance(m, ParallelSpec) else m
            if max(a.dim, a.vdim) > 1024:
                raise Unsupported(f"layer {i}: attention heads wider than 1024")
            if isinstance(m, ParallelSpec) and ops.delta_key_width(m.right.dim) is None:
                raise Unsupported(f"layer {i}: key width {m.right.dim} of the delta rule is above 512")
        self.layers: list[_Layer] = []
        self._places = self._place()

    # ---- cache geometry and scheduling hooks ------------------------------------------------------------------------
    @staticmethod
    def _value_heads(m: AttentionSpec, exchanged: bool) -> tuple[int, int]:
        """(cached value heads, their padded width)."""
        n = values_together(m.kv_heads, up8(m.vdim)) if exchanged else 1
        return m.kv_heads // n, n * up8(m.vdim)

    def _run_geometry(self, i: int) -> list:
        """Of one run of layer i: keys and values, (parallel mixers) the delta rule's state, the windows of both sublayers' convolutions."""
        lay, canon = self.stack.layers[i], WindowGeometry((self.taps - 1, self.hp))
        m, par = lay.mixer, isinstance(lay.mixer, ParallelSpec)
        a = m.left if par else m
        nv, dv = self._value_heads(a, par)
        return [KvGeometry(a.kv_heads, up8(a.dim), dv, nv), *([self._delta_geometry(m.right)] if par else []), canon,
                *([canon] if lay.mlp is not None else [])]

    def _place(self) -> list[tuple[int, int, int, int]]:
        """Per run: where in the pool its keys and values, delta state and convolution windows are."""
        out, at = [], 0
        for i in self.runs:
            par = int(isinstance(self.stack.layers[i].mixer, ParallelSpec))
            out.append((at, at + 1, at + 1 + par, at + 2 + par))
            at += len(self._run_geometry(i))
        return out

    def kv_geometry(self) -> list:
        return [g for i in self.runs for g in self._run_geometry(i)]

    def decode_splits(self, batch: int, max_kv: int) -> tuple[int, ...]:
        """KV splits per layer: a window (plus the rest of its first tile) is all that a layer reads."""
        def splits(m) -> int:
            a, par = (m.left, True) if isinstance(m, ParallelSpec) else (m, False)
            keys, (nv, dv) = min(max_kv, a.window + 63) if a.window else max_kv, self._value_heads(a, par)
            if par and self.dtype == torch.bfloat16 and ops.exchange_decode_fits(a.heads, a.kv_heads, up8(a.dim), nv, dv):
                want, s = min(148 // batch, keys // 64, 32), 1       # one CTA per SM, four pages each at least
                while s * 2 <= want:
                    s *= 2
                return s
            return splits_for(batch, a.kv_heads * (nv if par else 1), keys)
        return tuple(splits(lay.mixer) for lay in self.stack.layers)

    @staticmethod
    def _rotation(m: AttentionSpec) -> tuple[int, float] | None:
        return (m.rot_dims, m.rot_base) if m.rot_dims else None

    def rotations(self) -> set[tuple[int, float]]:
        mixers = [m.left if isinstance(m, ParallelSpec) else m for m in (lay.mixer for lay in self.stack.layers)]
        return {self._rotation(m) for m in mixers} - {None}

    # ---- weights ------------------------------------------------------------------------------------------------------
    def load_state_dict(self, weights: dict[str, torch.Tensor]) -> "NafelixGpu":
        return self._build(lambda name, *shape: self.tensor(weights, name, *shape))

    def init_random(self, seed: int = 0, std: float = 0.02) -> "NafelixGpu":
        """Random weights generated on the device (benchmarks)."""
        g = torch.Generator(device=self.device).manual_seed(seed)

        def rnd(name: str, *shape: int) -> torch.Tensor:
            last = name.rsplit(".", 1)[-1]
            if last.startswith("norm") or name.endswith((".left.out", ".right.out")):
                return torch.ones(shape, device=self.device)
            if last in ("mix", "talk") and len(shape) == 2 and shape[0] == shape[1]:
                return torch.eye(shape[0], device=self.device)
            if ".hc" in name:
                return torch.full(shape, 1.0 / shape[0], device=self.device)
            return torch.empty(shape, dtype=self.dtype, device=self.device).normal_(0.0, std, generator=g)
        return self._build(rnd)

    def _build(self, get) -> "NafelixGpu":
        W, V, S = self.width, self.cfg.vocab_size, self.streams

        def norm(name: str, factor: float = 1.0) -> NormWeights:
            return NormWeights(self._fp32(get(name, W).to(self.device, torch.float32) * factor, self.hp))

        def sublayer(L: str, n: int) -> _Sublayer:
            q = f"{L}hc{n}."
            return _Sublayer(norm(f"{L}norm{n}"), self._fp32(get(q + "in", S)), StreamMix(self._fp32(get(q + "mix", S, S)), self._fp32(get(q + "out", S))),
                             self._fp32(get(f"{L}canon{n}", W, self.taps).t(), self.hp))
        self.embed, self.head, self.final = self._mat(get("embed", V, W)), self._mat(get("head", V, W)), norm("final.norm")
        self.layers = []
        for i, spec in enumerate(self.stack.layers):
            L, m = f"l{i}.", spec.mixer
            p = L + "mix."
            if isinstance(m, ParallelSpec):
                rows, attention = self._attention(m.left, p + "left.", get, exchanged=True)
                more, delta = self._delta(m.right, p + "right.", get, sum(r.shape[0] for r in rows))
                lay = _Layer(torch.cat(rows + more), attention, sublayer(L, 1), delta=delta,
                             norms=(norm(p + "left.out", 0.5), norm(p + "right.out", 0.5)))
            else:
                rows, attention = self._attention(m, p, get, exchanged=False)
                bias = torch.cat([self._bias(get(f"{p}{n}.b", h * d), h, d, order) for n, h, d, order in
                                  (("q", m.heads, m.dim, m.rot_dims), ("k", m.kv_heads, m.dim, m.rot_dims), ("v", m.kv_heads, m.vdim, 0))])
                w_in = torch.cat(rows)
                lay = _Layer(w_in, attention, sublayer(L, 1), torch.nn.functional.pad(bias, (0, w_in.shape[0] - bias.numel())))
            if spec.mlp is not None:
                lay.ff, lay.ffn = self._feed_forward(spec.mlp, L + "mlp.", get), sublayer(L, 2)
            self.layers.append(lay)
        return self

    def _attention(self, m: AttentionSpec, p: str, get, exchanged: bool) -> tuple[list[torch.Tensor], _Attention]:
        """(projections q, k, v, gate; the rest)."""
        W, H, G, D, E, dk, vp = self.width, m.heads, m.kv_heads, m.dim, m.vdim, up8(m.dim), up8(m.vdim)
        order = torch.tensor(half_pairs(D, m.rot_dims))

        def turned(name: str, n: int) -> torch.Tensor:
            t = get(p + name, n * D, W)
            return self._heads(t.view(n, D, W)[:, order.to(t.device)], n, [(D, dk)])
        gate = self._heads(get(p + "g", H, W), 1, [(H, up8(H))]) if exchanged else self._heads(get(p + "g", H * E, W), H, [(E, vp)])
        nv, dv = self._value_heads(m, exchanged)
        a = _Attention(m, dk, dv, nv, self._fp32(get(p + "sink", H)), self._out(get(p + "o", W, H * E), H, E, vp), self._rotation(m))
        if exchanged:
            a.talk = ops.head_mix_weights(self._fp32(get(p + "talk", H, H)), G)
        else:
            a.unit = D
        return [turned("q", H), turned("k", G), self._heads(get(p + "v", G * E, W), G, [(E, vp)]), gate], a

    def _bias(self, b: torch.Tensor, n: int, d: int, rot: int) -> torch.Tensor:
        b = b.to(self.device, self.dtype).view(n, d)[:, torch.tensor(half_pairs(d, rot), device=self.device)]
        return torch.nn.functional.pad(b, (0, up8(d) - d)).reshape(-1)

    def _delta(self, m: HeadDeltaSpec, p: str, get, col: int) -> tuple[list[torch.Tensor], _Delta]:
        W, H, E, dp, vp, hb = self.width, m.heads, m.vdim, ops.delta_key_width(m.dim), up8(m.vdim), up8(m.heads)
        rows, conv = self._delta_inputs(m, p, get)
        col_b = 2 * m.kv_heads * dp + H * vp
        rows += [self._heads(get(p + n, H, W), 1, [(H, hb)]) for n in ("b", "a")] + [self._heads(get(p + "g", H * E, W), H, [(E, vp)])]
        w = DeltaWeights(H, m.kv_heads, m.dim, dp, E, vp, col_b, conv, self._fp32(get(p + "A_log", H)), self._fp32(get(p + "dt_bias", H)),
                         self._fp32(get(p + "norm", E), vp), head_decay=True, col_a=col_b + hb)
        return rows, _Delta(w, self._out(get(p + "o", W, H * E), H, E, vp), col, col_b + 2 * hb)

    def _feed_forward(self, f: DenseSpec | ExpertsSpec, p: str, get) -> _FeedForward:
        W, ff, fp = self.width, f.ff, up8(f.ff)
        if isinstance(f, DenseSpec):
            softplus = lambda z: math.log1p(math.exp(-abs(z))) + max(z, 0.0)   # noqa: E731
            a, b = (softplus(float(z)) for z in get(p + "act", 2).float().cpu())
            return _FeedForward(f, self._heads(get(p + "up", ff, W), 1, [(ff, fp)]), self._out(get(p + "down", W, ff), 1, ff, fp), (a, 0.5 + b))
        E = f.experts
        w = _FeedForward(f, torch.empty((E, 2 * fp, self.hp), dtype=self.dtype, device=self.device),
                         torch.empty((E, self.hp, fp), dtype=self.dtype, device=self.device),
                         router=self._heads(get(p + "router", E, W), 1, [(E, up8(E))]))
        for e in range(E):
            q = f"{p}e{e}."
            w.up[e] = self._pairs(get(q + "gate", ff, W), get(q + "up", ff, W))
            w.down[e] = self._out(get(q + "down", W, ff), 1, ff, fp)
        return w

    def weight_bytes(self) -> int:
        """Of one pass through the layers and the logits."""
        ts = [self.head]
        for lay in self.layers:
            ts += [lay.w_in, lay.attention.o] + ([lay.delta.o] if lay.delta is not None else [])
            if lay.ff is not None:
                ts += [t for t in (lay.ff.up, lay.ff.down, lay.ff.router) if t is not None]
        return sum(t.nbytes for t in ts)

    # ---- forward --------------------------------------------------------------------------------------------------------
    rows_per_expert_small = 4      # as for the other routed experts: above it the padded tiles win

    def _attend(self, a: _Attention, proj: torch.Tensor, gate: torch.Tensor, inp: StepInputs, kv, splits: int) -> torch.Tensor:
        """Attention up to its output projection; gate: logits per head (exchanged weights) or per output element."""
        m, T, (kc, vc), (nq, nk, nv) = a.spec, proj.shape[0], kv, a.cols
        ops.row_rope_kv_write(proj, inp.positions, inp.slot_mapping, kc, vc, m.heads, m.kv_heads, a.dk, v_col=nq + nk,
                              rope=self._rope[a.rope] if a.rope else None, unit=a.unit, eps=self.cfg.rms_norm_eps)
        fresh = None
        if inp.fresh_prefill and inp.cu_q is not None:
            fresh = (proj[:, nq:nq + nk].view(T, m.kv_heads, a.dk), proj[:, nq + nk:nq + nk + nv].view(T, a.value_heads, a.dv))
        self.launches += 2
        kw = dict(cu_q=inp.cu_q, max_q_len=inp.max_q_len, scale=m.scale, window=m.window, sink=a.sink, gate=gate, decode=inp.decode,
                  num_splits=splits, fresh_kv=fresh)
        q = proj[:, :nq].view(T, m.heads, a.dk)
        if a.talk is None:
            return ops.chunk_attention(q, kc, vc, inp.block_table, inp.kv_lens, **kw)
        self.launches += 1
        return ops.exchange_attention(q, kc, vc, inp.block_table, inp.kv_lens, talk=a.talk, **kw)

    def _mixer(self, lay: _Layer, h: torch.Tensor, inp: StepInputs, kv: list, place: tuple[int, ...], splits: int) -> HyperBranch:
        a, m = lay.attention, lay.attention.spec
        proj = self._linear(h, lay.w_in, bias=lay.b_in)
        g = sum(a.cols)
        gate = proj[:, g:g + (m.heads if a.talk is not None else m.heads * a.dv)]
        left = self._linear(self._attend(a, proj, gate, inp, kv[place[0]], splits), a.o)
        if lay.delta is None:
            return HyperBranch(left)
        d = lay.delta
        w, buf, (state, window) = d.weights, proj[:, d.col:], kv[place[1]]
        right = ops.head_delta(buf, buf[:, d.col_gate:d.col_gate + w.heads * w.vp], w, self.cfg.rms_norm_eps, state, window, inp.state_slots,
                               inp.positions, cu_q=inp.cu_q, max_q_len=inp.max_q_len)
        self.launches += 3
        return HyperBranch(left, lay.norms[0], self._linear(right, d.o), lay.norms[1])

    def _ffn(self, ff: _FeedForward, h: torch.Tensor) -> HyperBranch:
        T, f, fast = h.shape[0], ff.spec, self.dtype == torch.bfloat16
        if isinstance(f, DenseSpec):
            return HyperBranch(self._linear(self._linear(h, ff.up, act="xielu", act_params=ff.act), ff.down))
        logits = self._linear(h, ff.router, torch.float32)
        spread = fast and T * f.top > self.rows_per_expert_small * f.experts
        plan, rows = ops.logits_routing(logits, f.experts, f.top, rows=h if spread else None, renorm=True)
        y = ops.routed_gated_ffn(rows if spread else h, ff.up, ff.down, plan, "clamped", f.limit)
        self.launches += 3 if T <= 128 and not spread else 4 if fast and not spread else 5
        return HyperBranch(RoutedRows(y, plan.dest, plan.weights))

    def forward_hidden(self, inp: StepInputs, kv: list, *, tap=None) -> torch.Tensor:
        """Runs all layer runs; kv is `LayeredKvPool.data`. Returns final-normed rows [T | len(logits_rows), Hp]. `tap` (debugging) is
        called with the sum of the streams after every run."""
        if inp.embed_rows is not None or inp.rope_table is not None or inp.deepstack is not None:
            raise Unsupported("Nafelix takes token ids only")
        T, hp, dev, S, eps = inp.input_ids.numel(), self.hp, self.device, self.streams, self.cfg.rms_norm_eps
        single = inp.cu_q is None and inp.max_q_len == 1
        self.launches = 1
        x = ops.stream_embed(inp.input_ids, self.embed)           # all streams are alike until the first join
        joined = torch.empty((T, S, hp), dtype=torch.float32, device=dev)
        pending: tuple[HyperBranch, StreamMix] | None = None

        def advance(norm: NormWeights | None = None, read: torch.Tensor | None = None, **kw) -> torch.Tensor | None:
            """Joins the pending branch to the streams and writes what the next sublayer (or the logits) reads, normed."""
            nonlocal x, pending
            self.launches += 1
            out = torch.empty((T, hp), dtype=self.dtype, device=dev) if norm is not None else None
            branch, join = pending or (None, None)
            ops.hyper_step(x, S, self.width, eps, branch=branch, join=join, x_out=joined if branch is not None else None, read=read, norm=norm,
                           out=out, **kw)
            if branch is not None:
                x, pending = joined, None
            return out

        def enter(sub: _Sublayer, window: torch.Tensor) -> torch.Tensor:
            conv = ShortConv(sub.conv, window)
            if single:
                return advance(sub.norm, sub.read, conv=conv, slots=inp.state_slots, positions=inp.positions)
            self.launches += 1
            return ops.short_conv(advance(sub.norm, sub.read), conv, inp.state_slots, inp.positions, cu_q=inp.cu_q, max_q_len=inp.max_q_len)
        splits = inp.attn_splits if isinstance(inp.attn_splits, tuple) else (inp.attn_splits,) * len(self.layers)
        for i, place in zip(self.runs, self._places):
            lay = self.layers[i]
            pending = self._mixer(lay, enter(lay.mixer, kv[place[2]][0]), inp, kv, place, splits[i]), lay.mixer.join
            if lay.ff is not None:
                pending = self._ffn(lay.ff, enter(lay.ffn, kv[place[3]][0])), lay.ffn.join
            if tap is not None:
                advance()
                tap(x.sum(1)[:, :self.width])
        if inp.logits_rows is None:
            return advance(self.final)
        if pending is not None:
            advance()
        out = torch.empty((inp.logits_rows.numel(), hp), dtype=self.dtype, device=dev)
        self.launches += 1
        return ops.hyper_step(x, S, self.width, eps, norm=self.final, out=out, rows=inp.logits_rows)
