"""Zobunex decoder on sm_100a kernels: layers listed one by one in the config, a range of them run several times in a row.

Per layer run (x is the fp32 residual stream, LN a layer norm with bias):

    x += LN1b(attention(LN1(x)))      x += LN2b(experts(LN2(x)))

* attention: grouped heads with a q / k width and a v width of their own, interleaved rotary positions on the leading
  dimensions, keys limited to the query's own chunk of positions, and a learned sink in the softmax denominator;
* experts: every token id's experts come from a table (equal weights, no router), each expert is down(relu(up x)^2);
* loop: before each pass over the looped range x <- W [x; x0], x0 the embedding rows; every pass has its own cache;
* logits: final LN, then the embedding table, times a constant.

How that maps onto the device: the stream stays in fp32 and is touched by one kernel per sublayer, which norms the branch,
adds it, and norms the sum for the next consumer (`ops.stream_norm`); projections are the framework's bf16 GEMMs; one launch
at the start of a step plans the expert routing of every layer, because it depends on the token ids only; large steps store
the normed rows straight into the expert-sorted buffer of the grouped tcgen05 GEMM, small ones run a weight-streaming grouped
kernel; attention reads the paged cache (prefill on the tcgen05 kernel, decode on the TMA-fed split-KV kernel). A float32
instance runs everything in true 32-bit on the plain kernels, for numerical checks.

Widths that are not multiples of eight are padded with zero rows / columns at load time, which changes no result."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..contracts.errors import LoadError, Unsupported
from ..engine.kv_pool import KvGeometry
from ..ops import Branch, NormWeights
from ..parallel.comm import Communicator
from .config import AttentionSpec, ExpertsSpec, ModelConfig
from .llama import StepInputs, splits_for
from .stack import StackDecoder, up8 as _up8


@dataclass
class _Layer:
    spec: AttentionSpec
    dk: int                     # padded head widths
    dv: int
    norm1: NormWeights
    norm1b: NormWeights
    qkv: torch.Tensor           # [(H + G) * dk + G * dv, Hp]
    sink: torch.Tensor          # fp32 [H]
    o: torch.Tensor             # [Hp, H * dv]
    rope: tuple[int, float]
    experts: ExpertsSpec | None = None
    norm2: NormWeights | None = None
    norm2b: NormWeights | None = None
    up: torch.Tensor | None = None       # [E, Fp, Hp]
    down: torch.Tensor | None = None     # [E, Hp, Fp]
    table: tuple[tuple[int, int], int] | None = None   # (routing group, index in it)


class ZobunexGpu(StackDecoder):
    name = "Zobunex"

    def __init__(self, cfg: ModelConfig, comm: Communicator | None = None, device: torch.device | None = None,
                 dtype: torch.dtype = torch.bfloat16):
        super().__init__(cfg, comm, device, dtype)
        self.runs = self.stack.runs()
        self.loops = self.stack.loop is not None
        self.layers: list[_Layer] = []
        self.tables: dict[tuple[int, int], torch.Tensor] = {}   # (experts, top) -> int32 [layers of the group, vocab, top]
        self.loop_in = None

    # ---- cache geometry and scheduling hooks ----------------------------------------------------------------
    def kv_geometry(self) -> list[KvGeometry]:
        lays = self.stack.layers
        return [KvGeometry(lays[i].mixer.kv_heads, _up8(lays[i].mixer.dim), _up8(lays[i].mixer.vdim)) for i, _ in self.runs]

    def decode_splits(self, batch: int, max_kv: int) -> tuple[int, ...]:
        """KV splits per layer: a chunked layer never reads more than one chunk (plus the rest of its first tile)."""
        return tuple(splits_for(batch, m.kv_heads, min(max_kv, m.chunk + 63) if m.chunk else max_kv)
                     for m in (lay.mixer for lay in self.stack.layers))

    def rotations(self) -> set[tuple[int, float]]:
        return {(lay.mixer.rot_dims, lay.mixer.rot_base) for lay in self.stack.layers}

    # ---- weights ----------------------------------------------------------------------------------------------
    def load_state_dict(self, weights: dict[str, torch.Tensor]) -> "ZobunexGpu":
        W, V = self.width, self.cfg.vocab_size

        def get(name: str, *shape: int) -> torch.Tensor:
            return self.tensor(weights, name, *shape)

        def norm(name: str) -> NormWeights:
            return self._norm(get(name, W), get(name + ".b", W))

        self.embed = self._mat(get("embed", V, W))
        self.final = norm("final.norm")
        if self.loops:
            self.loop_in = self._loop_matrix(get("loop.in", W, 2 * W))
        self.layers, tables = [], {}
        for i, spec in enumerate(self.stack.layers):
            m, p = spec.mixer, f"l{i}.mix."
            lay = self._attention_layer(m, norm(f"l{i}.norm1"), norm(f"l{i}.norm1b"), get(p + "q", m.heads * m.dim, W),
                                        get(p + "k", m.kv_heads * m.dim, W), get(p + "v", m.kv_heads * m.vdim, W),
                                        get(p + "sink", m.heads), get(p + "o", W, m.heads * m.vdim))
            if spec.mlp is not None:
                e, p = spec.mlp, f"l{i}.mlp."
                lay.norm2, lay.norm2b = norm(f"l{i}.norm2"), norm(f"l{i}.norm2b")
                table = get(p + "table", V, e.top)
                if table.is_floating_point() or int(table.min()) < 0 or int(table.max()) >= e.experts:
                    raise LoadError(f"tensor {p}table must hold expert numbers below {e.experts}")
                self._set_experts(lay, e, [get(f"{p}e{x}.up", e.ff, W) for x in range(e.experts)],
                                  [get(f"{p}e{x}.down", W, e.ff) for x in range(e.experts)], table, tables)
            self.layers.append(lay)
        self._stack_tables(tables)
        return self

    def init_random(self, seed: int = 0, std: float = 0.02) -> "ZobunexGpu":
        """Random weights generated on the device (benchmarks)."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        W, V = self.width, self.cfg.vocab_size

        def rnd(*shape: int) -> torch.Tensor:
            return torch.empty(shape, dtype=self.dtype, device=self.device).normal_(0.0, std, generator=g)

        def norm() -> NormWeights:
            return self._norm(torch.ones(W), torch.zeros(W))

        self.embed, self.final = self._mat(rnd(V, W)), norm()
        if self.loops:
            self.loop_in = self._loop_matrix(rnd(W, 2 * W))
        self.layers, tables = [], {}
        for spec in self.stack.layers:
            m, e = spec.mixer, spec.mlp
            lay = self._attention_layer(m, norm(), norm(), rnd(m.heads * m.dim, W), rnd(m.kv_heads * m.dim, W),
                                        rnd(m.kv_heads * m.vdim, W), rnd(m.heads), rnd(W, m.heads * m.vdim))
            if e is not None:
                lay.norm2, lay.norm2b = norm(), norm()
                table = torch.rand((V, e.experts), generator=g, device=self.device).topk(e.top, dim=1).indices
                self._set_experts(lay, e, rnd(e.experts, e.ff, W), rnd(e.experts, W, e.ff), table, tables)
            self.layers.append(lay)
        self._stack_tables(tables)
        return self

    def _norm(self, w: torch.Tensor, b: torch.Tensor) -> NormWeights:
        return NormWeights(self._fp32(w, self.hp), self._fp32(b, self.hp))

    def _loop_matrix(self, w: torch.Tensor) -> torch.Tensor:
        W, out = self.width, torch.zeros((self.hp, 2 * self.hp), dtype=self.dtype, device=self.device)
        out[:W, :W] = w[:, :W].to(self.device, self.dtype)
        out[:W, self.hp:self.hp + W] = w[:, W:].to(self.device, self.dtype)
        return out

    def _attention_layer(self, m: AttentionSpec, norm1, norm1b, q, k, v, sink, o) -> _Layer:
        dk, dv = _up8(m.dim), _up8(m.vdim)
        pad = torch.nn.functional.pad

        def heads(t: torch.Tensor, n: int, d: int, dp: int) -> torch.Tensor:
            return pad(self._mat(t).view(n, d, self.hp), (0, 0, 0, dp - d)).reshape(n * dp, self.hp)
        qkv = torch.cat([heads(q, m.heads, m.dim, dk), heads(k, m.kv_heads, m.dim, dk), heads(v, m.kv_heads, m.vdim, dv)])
        o = pad(o.to(self.device, self.dtype).reshape(self.width, m.heads, m.vdim), (0, dv - m.vdim, 0, 0, 0, self.hp - self.width))
        return _Layer(m, dk, dv, norm1, norm1b, qkv.contiguous(), sink.to(self.device, torch.float32).contiguous(),
                      o.reshape(self.hp, m.heads * dv).contiguous(), (m.rot_dims, m.rot_base))

    def _set_experts(self, lay: _Layer, e: ExpertsSpec, up, down, table, tables: dict) -> None:
        fp = _up8(e.ff)
        lay.experts = e
        lay.up = torch.zeros((e.experts, fp, self.hp), dtype=self.dtype, device=self.device)
        lay.down = torch.zeros((e.experts, self.hp, fp), dtype=self.dtype, device=self.device)
        for x in range(e.experts):
            lay.up[x, :e.ff, :self.width] = up[x].to(self.device, self.dtype)
            lay.down[x, :self.width, :e.ff] = down[x].to(self.device, self.dtype)
        group = tables.setdefault((e.experts, e.top), [])
        lay.table = ((e.experts, e.top), len(group))
        group.append(table.to(self.device, torch.int32))

    def _stack_tables(self, tables: dict) -> None:
        self.tables = {k: torch.stack(v).contiguous() for k, v in tables.items()}

    def weight_bytes(self) -> int:
        ts = [self.embed] + ([self.loop_in] if self.loops else [])
        for lay in self.layers:
            ts += [lay.qkv, lay.o] + ([lay.up, lay.down] if lay.up is not None else [])
        return sum(t.nbytes for t in ts)

    # ---- forward ------------------------------------------------------------------------------------------------
    def _route(self, ids: torch.Tensor) -> dict:
        """Expert routing of every layer of this step. Steps with few rows per expert use dense segments (weight-streaming
        kernel), larger ones segments padded to the tile of the grouped tcgen05 GEMM."""
        T, plans = ids.numel(), {}
        for (experts, top), tables in self.tables.items():
            padded = self.dtype == torch.bfloat16 and T * top > self.rows_per_expert_small * experts
            plans[(experts, top)] = ops.table_routing(ids, tables, experts, padded=padded)
            self.launches += 1
        return plans

    rows_per_expert_small = 4      # measured on B200: above it the padded tiles win although most of their rows are empty

    def _attention(self, lay: _Layer, h: torch.Tensor, inp: StepInputs, kv, splits: int) -> torch.Tensor:
        m, T = lay.spec, h.shape[0]
        kc, vc = kv
        qkv = self._linear(h, lay.qkv)
        cos, sin = self._rope[lay.rope]
        ops.rope_kv_write(qkv, inp.positions, inp.slot_mapping, cos, sin, kc, vc, m.heads, m.kv_heads, lay.dk,
                          rot_dim=m.rot_dims, interleaved=True, block_size=kc.shape[2], v_dim=lay.dv)
        nq, nk = m.heads * lay.dk, m.kv_heads * lay.dk
        fresh = None
        if inp.fresh_prefill and inp.cu_q is not None:
            fresh = (qkv[:, nq:nq + nk].view(T, m.kv_heads, lay.dk), qkv[:, nq + nk:].view(T, m.kv_heads, lay.dv))
        self.launches += 2
        a = ops.chunk_attention(qkv[:, :nq].view(T, m.heads, lay.dk), kc, vc, inp.block_table, inp.kv_lens, cu_q=inp.cu_q,
                                max_q_len=inp.max_q_len, scale=m.scale, chunk=m.chunk, sink=lay.sink, decode=inp.decode,
                                num_splits=splits, fresh_kv=fresh)
        return self._linear(a, lay.o)

    def forward_hidden(self, inp: StepInputs, kv: list, *, tap=None) -> torch.Tensor:
        """Runs all layer runs; kv is `LayeredKvPool.data`. Returns final-normed rows [T | len(logits_rows), Hp], already
        carrying the logit scale. `tap` (debugging) is called with a copy of the residual stream after every run."""
        if inp.embed_rows is not None or inp.rope_table is not None or inp.deepstack is not None:
            raise Unsupported("Zobunex takes token ids only")
        T, hp, dev, eps = inp.input_ids.numel(), self.hp, self.device, self.cfg.rms_norm_eps
        self.launches = 1
        plans = self._route(inp.input_ids)
        cat = torch.empty((T, 2 * hp), dtype=self.dtype, device=dev) if self.loops else None     # [x; x0] of the loop
        halves = [] if cat is None else [cat[:, hp:], cat[:, :hp]] if self.runs[0][1] else [cat[:, hp:]]
        x = ops.stream_embed(inp.input_ids, self.embed, copies=halves)
        splits = inp.attn_splits if isinstance(inp.attn_splits, tuple) else (inp.attn_splits,) * len(self.layers)
        pending: Branch | None = None

        def advance(norm: NormWeights | None, out: torch.Tensor | None, **kw) -> torch.Tensor | None:
            """Joins the pending branch to the stream and writes the normed stream (the stream itself without `norm`)."""
            nonlocal pending
            b, pending = pending, None
            self.launches += 1
            return ops.stream_norm(x, self.width, eps, branch=b, norm=norm, out=out, **kw)

        for r, (i, enter) in enumerate(self.runs):
            lay = self.layers[i]
            if enter:
                if r > 0:
                    advance(None, cat[:, :hp])
                self._linear(cat, self.loop_in, torch.float32, out=x)
            h = advance(lay.norm1, torch.empty((T, hp), dtype=self.dtype, device=dev))
            pending = Branch(self._attention(lay, h, inp, kv[r], splits[i]), lay.norm1b)
            if lay.experts is not None:
                top = lay.experts.top
                plan = plans[lay.table[0]][lay.table[1]]
                if plan.padded:
                    h = advance(lay.norm2, torch.empty((plan.rows, hp), dtype=self.dtype, device=dev), out_rows=plan.dest,
                                out_top=top)
                else:
                    h = advance(lay.norm2, torch.empty((T, hp), dtype=self.dtype, device=dev))
                self.launches += 2
                pending = Branch(ops.routed_ffn(h, lay.up, lay.down, plan, "relu2"), lay.norm2b, plan.dest, top, 1.0 / top)
            if tap is not None:
                advance(None, None)
                tap(x[:, :self.width].clone())
        scale = self.stack.logit_scale
        if inp.logits_rows is None:
            return advance(self.final, torch.empty((T, hp), dtype=self.dtype, device=dev), out_scale=scale)
        if pending is not None:
            advance(None, None)
        return advance(self.final, torch.empty((inp.logits_rows.numel(), hp), dtype=self.dtype, device=dev),
                       rows=inp.logits_rows, out_scale=scale)
