"""Rotalorn on the GPU against the plain float64 restatement in tests/rotalorn_reference.py: each mechanism alone, then whole
models in float32 and bfloat16 through the runner, the paged pool, the generation loops, the provider and the replay tool."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import rotalorn_reference as ref

pytestmark = pytest.mark.gpu
F = torch.float64
DTYPES = [torch.float32, torch.bfloat16]
# relative RMS error of logits / of one mechanism's output
TOL = {torch.float32: 2e-5, torch.bfloat16: 3e-2}
OP_TOL = {torch.float32: 1e-5, torch.bfloat16: 8e-3}


def rel(got, want):
    got, want = got.detach().double().cpu(), want.double().cpu()
    return float((got - want).square().mean().sqrt() / want.square().mean().sqrt().clamp_min(1e-12))


def rnd(*shape, seed=0, dtype=torch.float32, std=1.0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * std).to(dtype)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


# ---- embedding, stream, projections ----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(50, 7, 3), (1, 5, 9), (997, 1 << 20, 999983)])
def test_pair_embedding_finds_the_previous_token(dtype, buckets, mul_prev, mul_cur):
    """Portions of several sequences over shuffled pages, cut at page borders, alone and side by side, uniform and ragged."""
    from inference_b200 import ops

    V, W, Hp, bs = 5000, 22, 24, 4
    table, pairs = (torch.nn.functional.pad(rnd(n, W, seed=n, dtype=dtype), (0, Hp - W)) for n in (V, buckets + 1))
    toks = [torch.randint(0, V, (n,), generator=torch.Generator().manual_seed(n)).tolist() for n in (13, 9, 4)]
    blocks = [[7, 2, 9, 0], [5, 1, 8], [3]]
    pages = torch.full((10, bs), 4321, dtype=torch.int32, device="cuda")
    bt = torch.zeros((3, 6), dtype=torch.int32)
    for i, b in enumerate(blocks):
        bt[i, :len(b)] = torch.tensor(b)
    at = [0, 0, 0]
    for cut in ([4, 1, 0], [1, 3, 0], [1, 1, 2], [3, 0, 1], [1, 1, 1], [3, 3, 0]):
        live = [i for i in range(3) if cut[i]]
        pos = [p for i in live for p in range(at[i], at[i] + cut[i])]
        ids = [toks[i][p] for i in live for p in range(at[i], at[i] + cut[i])]
        slots = [blocks[i][p // bs] * bs + p % bs for i in live for p in range(at[i], at[i] + cut[i])]
        uniform = len({cut[i] for i in live}) == 1
        x = ops.stream_embed_pairs(torch.tensor(ids).cuda(), table.cuda(), pairs.cuda(), mul_prev, mul_cur, positions=i32(pos),
                                   slots=torch.tensor(slots).cuda(), tokens=pages, block_table=bt[live].cuda(),
                                   cu_q=None if uniform else i32([0] + [cut[i] for i in live]).cumsum(0).int(), num_seqs=len(live),
                                   max_q_len=max(cut))
        want = []
        for i in live:
            rows = ref.bigram_rows(toks[i], buckets, mul_prev, mul_cur)
            want += [table[toks[i][p]].float() + pairs[rows[p]].float() for p in range(at[i], at[i] + cut[i])]
            at[i] += cut[i]
        assert torch.equal(x.cpu(), torch.stack(want))
    assert at == [13, 9, 4]
    assert int((pages == 4321).sum()) == 40 - 26                 # nothing but the tokens' own slots was written


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,Hp,top", [(90, 96, 1), (144, 144, 3), (2048, 2048, 8), (5000, 5000, 2)])
def test_parallel_sublayers_join_the_stream(dtype, H, Hp, top):
    """x += y + sum_k weight_k row_k, then the layer norm of the sum."""
    from inference_b200 import ops

    T, eps, R = 5, 1e-2, 23
    pad = lambda t: torch.nn.functional.pad(t, (0, Hp - H)).cuda().contiguous()   # noqa: E731
    x, y, e, w, b = rnd(T, H, seed=1) + 3, rnd(T, H, seed=2, dtype=dtype), rnd(R, H, seed=3, dtype=dtype), rnd(H, seed=4), rnd(H, seed=5)
    rows = torch.stack([torch.randperm(R, generator=torch.Generator().manual_seed(t))[:top] for t in range(T)])
    share = rnd(T, top, seed=6).abs()
    joined = x.double() + y.double() + (e.double()[rows] * share.double()[..., None]).sum(1)
    gx, out = pad(x), torch.full((T, Hp), 9.0, device="cuda")
    ops.stream_norm(gx, H, eps, branch=ops.Branch(pad(y), None, extra=ops.RoutedRows(pad(e), rows.int().cuda(), share.cuda())),
                    norm=ops.NormWeights(pad(w), pad(b)), out=out)
    assert rel(gx[:, :H], joined) < 1e-6 and rel(out[:, :H], ref.layer_norm(joined, w.double(), b.double(), eps)) < 5e-6
    assert (out[:, H:] == 0).all() and (gx[:, H:] == 0).all()


@pytest.mark.parametrize("rot", [{"dims": 24, "base": 700.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 96}},
                                 {"dims": 64, "base": 1e4, "scaling": {"factor": 3.0, "low": 2.0, "high": 9.0, "original": 700.5}}, {"dims": 6, "base": 30.0}])
def test_rotation_tables(rot):
    from inference_b200.models.config import RopeScaling
    from inference_b200.models.rotalorn import RotalornGpu

    s = rot.get("scaling")
    key = (rot["dims"], rot["base"], RopeScaling(s["factor"], s["low"], s["high"], s["original"]) if s else None)
    m = RotalornGpu.__new__(RotalornGpu)
    m.max_positions, m._rope, m.device, m.rotations = 0, {}, torch.device("cuda"), lambda: {key}
    m.stack = type("S", (), {"layers": ()})
    m.ensure_rope(3000)
    f = torch.tensor(ref.frequencies(rot), dtype=F)
    ang = torch.arange(3000, dtype=F)[:, None] * f
    cos, sin = m._rope[key]
    assert float((cos.double().cpu() - ang.cos()).abs().max()) < 1e-7 and float((sin.double().cpu() - ang.sin()).abs().max()) < 1e-7
    if s:
        plain = torch.tensor(ref.frequencies({k: rot[k] for k in ("dims", "base")}), dtype=F)
        kinds = (f / plain)
        assert kinds.max() == 1 and abs(float(kinds.min()) - 1 / s["factor"]) < 1e-12 and ((kinds < 0.999) & (kinds > 1.001 / s["factor"])).any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,rot", [(6, 2, 40, 24), (1, 1, 10, 6), (16, 1, 64, 64), (2, 1, 136, 100), (32, 8, 128, 128)])
def test_whole_projection_norms_rotation_and_raw_values(dtype, H, G, D, rot):
    from inference_b200 import ops
    from inference_b200.models.latent_mixer import half_pairs

    T, dp, bs, eps, order = 5, (D + 7) // 8 * 8, 16, 1e-3, half_pairs(D, rot)
    q, k = rnd(T, H, D, seed=1, dtype=dtype) * 2, rnd(T, G, D, seed=2, dtype=dtype) * 0.3
    wq, wk = rnd(H * D, seed=3), rnd(G * D, seed=4)
    pos, slots = torch.tensor([0, 1, 40, 7, 63]), torch.tensor([35, 3, 16, -1, 47])
    spec = {"dims": rot, "base": 500.0}
    ang = torch.arange(64, dtype=F)[:, None] * torch.tensor(ref.frequencies(spec), dtype=F)
    lay = lambda t: torch.nn.functional.pad(t[..., order], (0, dp - D))            # noqa: E731
    nq, nk = H * dp, G * dp
    buf = torch.cat([lay(q).reshape(T, nq), lay(k).reshape(T, nk), torch.full((T, nk), 5.0, dtype=dtype)], 1).cuda()
    kc, vc = (torch.zeros((4, G, bs, dp), dtype=dtype, device="cuda") for _ in range(2))
    ops.row_rope_kv_write(buf, pos.int().cuda(), slots.cuda(), kc, vc, H, G, dp, v_col=nq + nk, rope=(ang.cos().float().cuda(), ang.sin().float().cuda()),
                          q_norm=lay(wq.view(H, D)).reshape(-1).cuda(), k_norm=lay(wk.view(G, D)).reshape(-1).cuda(), norm_counts=(H * D, G * D), eps=eps,
                          v_from_k=True, store_v=True)
    want = [ref.rotate_halves((ref.rms(t.double().reshape(T, -1), eps) * w.double()).view(T, -1, D), pos, spec) for t, w in ((q, wq), (k, wk))]
    back = lambda t, n: t.reshape(T, n, dp)[..., :D]                              # noqa: E731
    assert rel(back(buf[:, :nq], H), want[0][..., order]) < OP_TOL[dtype] and rel(back(buf[:, nq:nq + nk], G), want[1][..., order]) < OP_TOL[dtype]
    assert torch.equal(back(buf[:, nq + nk:], G).cpu(), k[..., order])
    for cache, w in ((kc, want[1]), (vc, k.double())):
        flat = cache.transpose(1, 2).reshape(-1, G, dp)
        for t in (0, 1, 2, 4):
            assert rel(flat[slots[t], :, :D], w[t][..., order]) < OP_TOL[dtype]
        assert int((flat != 0).any(-1).any(-1).sum()) == 4 and (flat[..., D:] == 0).all()
    # no norm, no rotation, values of their own width: only the caches are written
    kv = torch.cat([lay(k).reshape(T, nk), rnd(T, G * 24, seed=9, dtype=dtype)], 1).cuda()
    keep, vc = kv.clone(), torch.zeros((4, G, bs, 24), dtype=dtype, device="cuda")
    kc.zero_()
    ops.row_rope_kv_write(kv, pos.int().cuda(), slots.cuda(), kc, vc, 0, G, dp, v_col=nk)
    assert torch.equal(kv, keep)
    assert torch.equal(vc.transpose(1, 2).reshape(-1, G * 24)[35], kv[0, nk:]) and torch.equal(kc.transpose(1, 2).reshape(-1, nk)[47], kv[4, :nk])


# ---- feed-forward -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("act", ["gelu", "silu"])
def test_gated_activation_with_row_gate(dtype, act):
    from inference_b200 import ops

    T, ff = 5, 72
    g, u, z = rnd(T, ff, seed=1, dtype=dtype) * 3, rnd(T, ff, seed=2, dtype=dtype), rnd(T, 4, seed=3)
    want = (ref.gelu if act == "gelu" else ref.silu)(g.double()) * u.double()
    out = torch.zeros((T, ff + 16), dtype=dtype, device="cuda")
    pairs = torch.stack([g, u], -1).reshape(T, -1).cuda()
    ops.gated_act_mul(pairs, act, out=out[:, 8:8 + ff], paired=True)
    assert rel(out[:, 8:8 + ff], want) < OP_TOL[dtype] and (out[:, :8] == 0).all() and (out[:, 8 + ff:] == 0).all()
    ops.gated_act_mul(pairs, act, out=out[:, 8:8 + ff], paired=True, row_gate=z.cuda()[:, 2])
    assert rel(out[:, 8:8 + ff], want * torch.sigmoid(z[:, 2:3].double())) < OP_TOL[dtype]
    assert rel(ops.gated_act_mul(torch.cat([g, u], 1).cuda(), act), want) < OP_TOL[dtype]


@pytest.mark.parametrize("padded", [False, True])
@pytest.mark.parametrize("T,E,top", [(1, 8, 2), (7, 3, 3), (19, 40, 6), (128, 64, 8), (129, 5, 1), (700, 33, 4), (3, 100, 40), (2000, 8, 2)])
def test_routing_plans(T, E, top, padded):
    """Choice, order of ties, weights, and that the plan is a permutation into the experts' segments; twice, so that the counters are
    seen to clear."""
    from inference_b200 import ops

    for seed in (0, 1):
        z = rnd(T, E + 5, seed=seed) * 3
        z[:, E:] = 99.0                                        # not logits
        z[::3, :E] = z[::3, :E].round()                        # ties
        rows = rnd(T, 24, seed=5, dtype=torch.bfloat16).cuda() if padded else None
        plan, buf = ops.logits_routing(z.cuda(), E, top, rows=rows)
        e = torch.argsort(z[:, :E], dim=-1, descending=True, stable=True)[:, :top]
        w = torch.softmax(z[:, :E].double(), -1).gather(1, e)
        assert rel(plan.weights, w) < 1e-6
        start, dest = plan.offsets.cpu(), plan.dest.cpu().long()
        counts = torch.bincount(e.flatten(), minlength=E)
        step = (counts + 127) // 128 * 128 if padded else counts
        assert torch.equal(start[1:] - start[:-1], step.int())
        assert dest.flatten().unique().numel() == T * top
        assert ((dest >= start[e]) & (dest < start[e] + counts[e])).all()
        if padded:
            tiles = plan.tile_group.cpu()
            assert torch.equal(tiles[dest // 128].long(), e) and (tiles[int(start[-1]) // 128:] == -1).all()
            assert torch.equal(buf[dest.flatten().cuda()], rows.repeat_interleave(top, 0))
        else:
            assert torch.equal(plan.src.cpu()[dest].long(), torch.arange(T)[:, None].expand(-1, top))
            act = plan.active.cpu()
            assert sorted(act[act >= 0].tolist()) == counts.nonzero().flatten().tolist()
    assert (ops.moe._counters(torch.device("cuda")) == 0).all()


@pytest.mark.parametrize("dtype,padded", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
@pytest.mark.parametrize("T,E,top,W,ff", [(1, 4, 2, 96, 24), (40, 6, 3, 64, 56), (70, 3, 3, 256, 136)])
def test_routed_gated_experts(dtype, padded, T, E, top, W, ff):
    from inference_b200 import ops

    h, g, u, d = rnd(T, W, seed=1, dtype=dtype), *(rnd(E, ff, W, seed=s, std=W ** -0.5, dtype=dtype) for s in (2, 3)), rnd(E, W, ff, seed=4, std=ff ** -0.5, dtype=dtype)
    router = rnd(E, W, seed=5, std=2 * W ** -0.5)
    z = h.float() @ router.T
    e, w = ref.route(h.double(), router.double(), top)
    want = torch.zeros(T, W, dtype=F)
    for t in range(T):
        for j in range(top):
            x = int(e[t, j])
            want[t] += w[t, j] * (d[x].double() @ (ref.silu(g[x].double() @ h[t].double()) * (u[x].double() @ h[t].double())))
    plan, rows = ops.logits_routing(z.cuda(), E, top, rows=h.cuda() if padded else None)
    pairs = torch.stack([g, u], 2).reshape(E, 2 * ff, W).cuda()
    y = ops.routed_gated_ffn(rows if padded else h.cuda(), pairs, d.cuda(), plan, "silu")
    got = (y.float()[plan.dest.long()] * plan.weights[..., None]).sum(1)
    assert rel(got, want) < OP_TOL[dtype]


# ---- attention ----------------------------------------------------------------------------------------------------------
def _paged(rows, dtype, bs=16, seed=0):
    """Scatters each sequence's rows [n, heads, width] over shuffled pages [page, heads, bs, width]; unused rows hold large values."""
    need = [(len(r) + bs - 1) // bs for r in rows]
    perm = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    h, w = rows[0].shape[1:]
    cache, table = torch.full((len(perm), h, bs, w), 7.0).to(dtype), torch.zeros((len(rows), max(need) + 2), dtype=torch.int32)
    for s, r in enumerate(rows):
        for b in range(need[s]):
            table[s, b] = page = perm.pop()
            m = r[b * bs:(b + 1) * bs]
            cache[page, :, :len(m)] = m.transpose(0, 1).to(dtype)
    return cache.cuda(), table.cuda()


def _aligned(q, k, at, scale, score=20.0):
    """Makes the key at position `at` (of all heads' common direction) and the last query give a score that takes the whole softmax."""
    u = torch.nn.functional.normalize(rnd(q.shape[-1], seed=99), dim=0)
    if 0 <= at < len(k):
        k[at] = (u * 8).bfloat16().float()
    q[-1] = (u * score / (8 * scale)).bfloat16().float()


def _window_case(dtype, H, G, D, E, lens, q_lens, how, window, splits=1, plant=None, uniform=False, scale=None):
    """`plant`: distance of the standing-out key from the last query."""
    from inference_b200 import ops

    scale = D ** -0.5 if scale is None else scale
    b16 = lambda *s, seed: rnd(*s, seed=seed, dtype=torch.bfloat16).float()   # noqa: E731
    ks, vs = [b16(n, G, D, seed=10 + i) for i, n in enumerate(lens)], [b16(n, G, E, seed=30 + i) for i, n in enumerate(lens)]
    qs = [b16(n, H, D, seed=50 + i) for i, n in enumerate(q_lens)]
    if plant is not None:
        for q, k in zip(qs, ks):
            _aligned(q, k, len(k) - 1 - plant, scale)
    want = torch.cat([ref.softmax_attention(q.double(), k.double().repeat_interleave(H // G, 1), v.double().repeat_interleave(H // G, 1),
                                            torch.arange(len(k) - len(q), len(k)), scale, window) for q, k, v in zip(qs, ks, vs)])
    kc, table = _paged(ks, dtype)
    vc, _ = _paged(vs, dtype)
    q, fresh = torch.cat(qs).to(dtype).cuda(), None
    if how == "fresh":
        fresh = tuple(torch.cat(t).to(dtype).cuda() for t in (ks, vs))
    out = torch.full((len(q), H * E + 8), 3.0, dtype=dtype, device="cuda")
    ops.chunk_attention(q, kc, vc, table, i32(lens), cu_q=None if uniform else i32([0] + q_lens).cumsum(0).int(), max_q_len=max(q_lens), scale=scale,
                        window=window, decode=how == "decode", num_splits=splits, fresh_kv=fresh, out=out[:, :H * E],
                        kernel="simple" if how == "simple" else "auto")
    ops.check_status()
    assert (out[:, H * E:] == 3).all()
    return rel(out[:, :H * E].reshape(want.shape), want)


SHAPES = [(4, 2, 64, 64), (6, 2, 40, 24), (8, 1, 128, 128), (1, 1, 16, 8), (16, 1, 72, 96)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [1, 2, 17, 64, 129, 1000])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_window_attention(shape, window, how):
    lens = [401, 1, 130, 257, 37]
    q_lens = lens if how == "fresh" else [1] * 5 if how == "decode" else [150, 1, 2, 200, 20]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        for splits in (1, 2, 7) if how == "decode" else (1,):
            assert _window_case(dtype, *shape, lens, q_lens, how, window, splits, uniform=how == "decode") < OP_TOL[dtype]


@pytest.mark.parametrize("window", [1, 15, 16, 17, 40, 63, 64, 65, 128, 200])
@pytest.mark.parametrize("gap", [-1, 0, 1])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_keys_at_the_edge_of_a_window(window, gap, how):
    """A key that takes the whole softmax of the last query, one inside the edge, at it, or one outside."""
    lens = [385, 130, 64]
    q_lens = lens if how == "fresh" else [40, 1, 17] if how == "context" else [1, 2, 1]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        assert _window_case(dtype, 4, 2, 48, 32, lens, q_lens, how, window, 3, plant=window - 1 + gap) < OP_TOL[dtype]


@pytest.mark.parametrize("how", ["context", "decode"])
def test_window_attention_takes_a_few_tokens_each(how):
    assert _window_case(torch.bfloat16, 8, 4, 64, 64, [130, 66, 300], [4, 4, 4], how, 33, 2, uniform=True) < OP_TOL[torch.bfloat16]
    assert _window_case(torch.bfloat16, 8, 4, 64, 64, [130, 66, 300], [4, 1, 3], how, 33, 2) < OP_TOL[torch.bfloat16]
    assert _window_case(torch.bfloat16, 2, 1, 16, 16, [70, 66], [2, 2], how, 9, scale=-0.2) < OP_TOL[torch.bfloat16]      # plain kernel


def _diff_case(dtype, H, G, D, E, lens, q_lens, how, cap=20.0, coef=0.4, every=50, share=0.7, splits=1, plant=None, uniform=False, post=0.6):
    from inference_b200 import ops

    scale, eps = D ** -0.5, 1e-3
    dp, vp = (D + 7) // 8 * 8, (E + 7) // 8 * 8
    b16 = lambda *s, seed: rnd(*s, seed=seed, dtype=torch.bfloat16).float()   # noqa: E731
    ks, vs = [b16(n, G, 2, D, seed=10 + i) for i, n in enumerate(lens)], [b16(n, G, E, seed=30 + i) for i, n in enumerate(lens)]
    qs = [b16(n, H, 2, D, seed=50 + i) * 2 for i, n in enumerate(q_lens)]
    if plant is not None:                            # each map's last query has a key of its own
        for q, k in zip(qs, ks):
            for m in (0, 1):
                _aligned(q[:, :, m], k[:, :, m], (plant if plant >= 0 else len(k) + plant) + m, scale, 40.0)
    temp = ref.temperature(torch.arange(max(lens)), coef, every)
    want = []
    for q, k, v in zip(qs, ks, vs):
        pos = torch.arange(len(k) - len(q), len(k))
        q = q.double() * temp[pos][:, None, None, None]
        k, v = (t.double().repeat_interleave(H // G, 1) for t in (k, v))
        a1, a2 = (ref.softmax_attention(q[:, :, m], k[:, :, m], v, pos, scale, 0, cap) for m in (0, 1))
        want.append(ref.differ(a1, a2, share, 1 - post, eps))
    want = torch.cat(want)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))     # noqa: E731
    kc, table = _paged([pad(k, dp).reshape(len(k), G, 2 * dp) for k in ks], dtype)
    vc, _ = _paged([pad(v, vp) for v in vs], dtype)
    fresh = None
    if how == "fresh":
        fresh = pad(torch.cat(ks), dp).reshape(-1, G, 2 * dp).to(dtype).cuda(), pad(torch.cat(vs), vp).to(dtype).cuda()
    d = ops.Differential(share, post, eps, E, cap, temp.float().cuda() if coef else None)
    out = torch.full((sum(q_lens), H * vp + 8), 3.0, dtype=dtype, device="cuda")
    ops.chunk_attention(pad(torch.cat(qs), dp).to(dtype).cuda(), kc, vc, table, i32(lens), cu_q=None if uniform else i32([0] + q_lens).cumsum(0).int(),
                        max_q_len=max(q_lens), scale=scale, decode=how == "decode", num_splits=splits, diff=d, fresh_kv=fresh,
                        out=out[:, :H * vp], kernel="simple" if how == "simple" else "auto")
    ops.check_status()
    got = out[:, :H * vp].view(-1, H, vp)
    assert (out[:, H * vp:] == 3).all() and (got[..., E:] == 0).all()
    return rel(got[..., :E], want)


DIFF = [(4, 2, 32, 64), (4, 2, 24, 40), (3, 3, 64, 128), (8, 1, 64, 96), (2, 1, 9, 7), (1, 1, 5, 12), (16, 2, 16, 24)]


@pytest.mark.parametrize("shape", DIFF)
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_differential_attention(shape, how):
    lens = [401, 1, 130, 257, 37]
    q_lens = lens if how == "fresh" else [1] * 5 if how == "decode" else [150, 1, 2, 200, 20]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        for splits in (1, 2, 8, 16) if how == "decode" else (1,):
            assert _diff_case(dtype, *shape, lens, q_lens, how, splits=splits, uniform=how == "decode") < 2 * OP_TOL[dtype]


@pytest.mark.parametrize("cap,coef,every,share,post", [(0.0, 0.0, 1, 0.5, 1.0), (5.0, 1.5, 1, 1.3, 0.2), (100.0, 0.2, 1000, -0.4, 0.9), (30.0, 0.5, 7.5, 0.0, 0.5)])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_differential_constants(cap, coef, every, share, post, how):
    lens = [300, 70]
    q_lens = lens if how == "fresh" else [2, 2] if how == "decode" else [40, 3]
    dtype = torch.float32 if how == "simple" else torch.bfloat16
    assert _diff_case(dtype, 4, 2, 32, 48, lens, q_lens, how, cap, coef, every, share, 2, post=post, uniform=how == "decode") < 2 * OP_TOL[dtype]


@pytest.mark.parametrize("plant", [0, 14, 15, 16, 62, 63, 64, 127, 128, -3, -2])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_far_keys_of_both_maps(plant, how):
    """Each map's last query puts its whole weight on one key, far away, at page and tile borders, and next to itself."""
    lens = [385, 130, 64]
    q_lens = lens if how == "fresh" else [40, 1, 17] if how == "context" else [1, 2, 1]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        assert _diff_case(dtype, 4, 2, 32, 48, lens, q_lens, how, cap=50.0, splits=2, plant=plant) < 2 * OP_TOL[dtype]


# ---- latent attention with a window and low-rank queries ------------------------------------------------------------------
def _latent_weights(H, dim, rot, vdim, rank, window, dtype, q_rank=0, seed=0):
    from inference_b200 import ops

    up = lambda n, m: (n + m - 1) // m * m   # noqa: E731
    dn, rp, rk, vp, qk = up(dim, 16), up(rot, 8), up(rank, 64), up(vdim, 16), up(q_rank, 16)
    uk, uv = (rnd(H, d, rank, seed=seed + s, dtype=torch.bfloat16, std=rank ** -0.5) for s, d in ((1, dim), (2, vdim)))
    pad = lambda t, n: torch.nn.functional.pad(t, (0, rk - rank, 0, n - t.shape[1])).to(dtype).cuda()   # noqa: E731
    ku, vu = pad(uk, dn), pad(uv, vp)
    low = dict(q_rank=q_rank, qk=qk, q_norm=torch.nn.functional.pad(rnd(q_rank, seed=seed + 4), (0, qk - q_rank)).cuda()) if q_rank else {}
    w = ops.LatentWeights(H, dim, dn, rot, rp, rank, rk, vdim, vp, (dim + rot) ** -0.5, torch.nn.functional.pad(rnd(rank, seed=seed + 3), (0, rk - rank)).cuda(),
                          None, torch.cat([ku.reshape(H * dn, rk), vu.reshape(H * vp, rk)]), ku.transpose(1, 2).contiguous(), window=window, **low)
    return w, uk.double(), uv.double()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,rot,rank,q_rank", [(3, 40, 24, 96, 72), (1, 18, 6, 20, 11), (16, 128, 64, 512, 1536), (2, 16, 72, 600, 64)])
def test_low_rank_queries(dtype, H, dim, rot, rank, q_rank):
    """Both latents normed, the shared key part rotated and cached; the queries rotated in a launch of their own or with the key product."""
    from inference_b200 import ops

    w, uk, _ = _latent_weights(H, dim, rot, 16, rank, 0, dtype, q_rank)
    T, bs, eps = 5, 16, 1e-3
    pos, slots = torch.tensor([0, 1, 40, 7, 63]), torch.tensor([35, 3, 16, -1, 47])
    dq, low = rnd(T, q_rank, seed=1, dtype=dtype) * 2, rnd(T, rank + rot, seed=2, dtype=dtype) * 3
    proj = torch.zeros(T, w.col_gate + 8, dtype=dtype)
    proj[:, :q_rank], proj[:, w.col_c:w.col_c + rank] = dq, low[:, :rank]
    proj[:, w.col_c + w.rk:w.col_c + w.rk + rot], proj[:, w.col_gate:] = low[:, rank:], 2.0
    order = [j for i in range(rot // 2) for j in (i, i + rot // 2)]
    spec = {"dims": rot, "base": 300.0}
    unorder = lambda t: torch.empty_like(t).index_copy_(-1, torch.tensor(order), t)     # noqa: E731
    turn = lambda t: ref.rotate_halves(unorder(t.double()), pos, spec)[..., order]        # noqa: E731
    ang = torch.arange(64, dtype=F)[:, None] * torch.tensor(ref.frequencies(spec), dtype=F)
    cos, sin = ang.cos().float().cuda(), ang.sin().float().cuda()
    cache, buf = torch.zeros((4, bs, w.width), dtype=dtype, device="cuda"), proj.cuda()
    ops.latent_prep(buf, w, eps, cos, sin, pos.int().cuda(), slots.cuda(), cache)
    c = ref.rms(low[:, :rank].double(), eps) * w.norm[:rank].double().cpu()
    kr = turn(low[:, None, rank:])[:, 0]
    assert rel(buf[:, :q_rank], ref.rms(dq.double(), eps) * w.q_norm[:q_rank].double().cpu()) < OP_TOL[dtype] and (buf[:, q_rank:w.qk] == 0).all()
    assert rel(buf[:, w.col_c:w.col_c + rank], c) < OP_TOL[dtype] and (buf[:, w.col_gate:] == 2).all()
    flat = cache.view(-1, w.width)
    for t in (0, 1, 2, 4):
        assert rel(flat[slots[t], :rank], c[t]) < OP_TOL[dtype] and rel(flat[slots[t], w.rk:w.rk + rot], kr[t]) < OP_TOL[dtype]
    assert int((flat != 0).any(-1).sum()) == 4
    q = torch.zeros(T, H, w.dn + w.rp, dtype=dtype)
    q[..., :dim], q[..., w.dn:w.dn + rot] = rnd(T, H, dim, seed=6, dtype=dtype), rnd(T, H, rot, seed=7, dtype=dtype)
    want = turn(q[..., w.dn:w.dn + rot])
    gq, q_abs = q.view(T, -1).cuda(), torch.zeros((3, H, w.width), dtype=dtype, device="cuda")
    ops.rotate_queries(gq, w, cos, sin, pos.int().cuda(), q_abs, i32([2, -1, 0, 1, -1]))
    out = gq.view(T, H, -1)
    assert rel(out[..., w.dn:w.dn + rot], want) < OP_TOL[dtype] and torch.equal(out[..., :w.dn].cpu(), q[..., :w.dn])
    for row, t in enumerate((2, 3, 0)):
        assert rel(q_abs[row, :, w.rk:w.rk + rot], want[t]) < OP_TOL[dtype]
    if dtype == torch.bfloat16:
        q_abs = torch.full((T, H, w.width), 5.0, dtype=dtype, device="cuda")
        ops.head_product(q.cuda()[..., :w.dn], w.uk_t, q_abs[..., :w.rk],
                         rotate=ops.QueryRotation(cos, sin, pos.int().cuda(), w.dn, w.rot, w.rp, w.rc))
        assert rel(q_abs[..., w.rk:w.rk + rot], want) < OP_TOL[dtype] and (q_abs[..., w.rk + rot:] == 0).all()
        assert rel(q_abs[..., :rank], torch.einsum("thd,hdr->thr", q[..., :dim].double(), uk)) < OP_TOL[dtype]


def _latent_window_case(dtype, H, dim, rot, vdim, rank, lens, q_lens, how, window, splits=1, plant=None, listed=None):
    from inference_b200 import ops

    w, uk, uv = _latent_weights(H, dim, rot, vdim, rank, window, dtype)
    b16 = lambda *s, seed: rnd(*s, seed=seed, dtype=torch.bfloat16).float()   # noqa: E731
    cs, krs = [b16(n, rank, seed=10 + i) for i, n in enumerate(lens)], [b16(n, rot, seed=30 + i) for i, n in enumerate(lens)]
    qs = [b16(n, H, dim + rot, seed=50 + i) for i, n in enumerate(q_lens)]
    if plant is not None:
        for q, kr in zip(qs, krs):
            _aligned(q[..., dim:], kr, len(kr) - 1 - plant, w.scale)
    gate, want = rnd(sum(q_lens), H, seed=8, dtype=torch.bfloat16), []
    for c, kr, q in zip(cs, krs, qs):
        k, v = ref.latent_keys_values(c.double(), kr.double(), uk.reshape(-1, rank), uv.reshape(-1, rank), H)
        want.append(ref.softmax_attention(q.double(), k, v, torch.arange(len(c) - len(q), len(c)), w.scale, window))
    want = torch.cat(want) * torch.sigmoid(gate.double())[..., None]
    rows = []
    for c, kr in zip(cs, krs):
        r = torch.zeros(len(c), 1, w.width)
        r[:, 0, :rank], r[:, 0, w.rk:w.rk + rot] = c, kr
        rows.append(r)
    cache, table = _paged(rows, dtype)
    cache = cache[:, 0].contiguous()
    T = sum(q_lens)
    q = torch.zeros(T, H, w.dn + w.rp)
    q[..., :dim], q[..., w.dn:w.dn + rot] = torch.cat(qs)[..., :dim], torch.cat(qs)[..., dim:]
    q, g, out = q.to(dtype).cuda(), gate.to(dtype).cuda(), torch.zeros((T, H, w.vp), dtype=dtype, device="cuda")
    cu, keep = i32([0] + q_lens).cumsum(0).int(), slice(None)
    if how in ("decode", "simple"):
        q_abs = torch.empty((T, H, w.width), dtype=dtype, device="cuda")
        q_abs[..., w.rk:] = torch.nn.functional.pad(q[..., w.dn:], (0, w.rc - w.rp))
        ops.head_product(q[..., :w.dn], w.uk_t, q_abs[..., :w.rk])
        kw = dict(cu_q=cu, max_q_len=max(q_lens))
        lat = ops.latent_decode(q_abs, cache, table, i32(lens), w, num_splits=splits, **kw) if how == "decode" else \
            ops.latent_attention_simple(q_abs, cache, table, i32(lens), w, **kw)
        ops.head_product(lat, w.uv, out, gate=g, sink=w.sink)
    else:
        ids, kw, flat = listed or list(range(len(lens))), {}, torch.cat(rows)[:, 0].to(dtype).cuda()
        if how == "context":                       # only the key rows that some query sees
            first = [max(0, lens[i] - q_lens[i] - window + 1) for i in ids]
            n = [lens[i] - f for i, f in zip(ids, first)]
            cu_k = i32([0] + n).cumsum(0).int()
            flat = ops.latent_gather(cache, table, cu_k, sum(n), i32(ids), i32(first))
            assert torch.equal(flat.cpu(), torch.cat([rows[i][f:, 0] for i, f in zip(ids, first)]).to(dtype))
            kw = dict(seqs=i32(ids), cu_k=cu_k)
            starts = [0] + torch.tensor(q_lens).cumsum(0).tolist()
            keep = [t for i in ids for t in range(starts[i], starts[i + 1])]
        kv = ops.gemm_bf16(flat[:, :w.rk], w.ukv)
        ops.latent_prefill(q.view(T, -1), kv, flat[:, w.rk:w.rk + w.rp], w, out.view(T, -1), cu_q=cu, max_q_len=max(q_lens[i] for i in ids), gate=g, **kw)
    ops.check_status()
    return rel(out[keep][..., :vdim], want[keep])


LATENT = [(4, 64, 16, 64, 128), (3, 40, 24, 56, 96), (16, 128, 64, 128, 512), (20, 32, 32, 48, 192), (1, 18, 6, 14, 20)]


@pytest.mark.parametrize("shape", LATENT)
@pytest.mark.parametrize("window", [1, 2, 40, 64, 129, 1000])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_latent_window(shape, window, how):
    lens = [401, 1, 130, 257, 37]
    q_lens = lens if how == "fresh" else [5, 1, 7, 2, 16] if how == "decode" else [150, 1, 2, 200, 20]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        for splits in (1, 2, 7) if how == "decode" else (1,):
            assert _latent_window_case(dtype, *shape, lens, q_lens, how, window, splits) < OP_TOL[dtype]
    if how == "context":
        assert _latent_window_case(torch.bfloat16, *shape, lens, q_lens, how, window, listed=[3, 0, 4]) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("window", [1, 16, 40, 63, 64, 65, 128, 200])
@pytest.mark.parametrize("gap", [-1, 0, 1])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_latent_keys_at_the_edge_of_a_window(window, gap, how):
    lens = [385, 130, 64]
    q_lens = lens if how == "fresh" else [40, 1, 17] if how == "context" else [1, 2, 1]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        assert _latent_window_case(dtype, 4, 48, 16, 32, 64, lens, q_lens, how, window, 3, plant=window - 1 + gap) < OP_TOL[dtype]


# ---- whole models ----------------------------------------------------------------------------------------------------
_CACHE: dict = {}


def _model(name):
    if name not in _CACHE:
        cfg = ref.MODELS[name]()
        _CACHE[name] = (cfg, ref.random_weights(cfg, seed=ord(name)), {})
    return _CACHE[name]


def _tokens(name, n, seed=0):
    return torch.randint(0, _model(name)[0]["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _want(name, tokens):
    cfg, w, memo = _model(name)
    key = tuple(tokens)
    if key not in memo:
        memo[key] = ref.run(cfg, w, tokens)
    return memo[key]


def _sure(name, tokens, gap=0.15):
    """Rows whose experts are no close call: rounding h to bf16 cannot choose others."""
    cfg, w, _ = _model(name)
    m = []
    ref.run(cfg, w, tokens, m)
    return torch.stack(m).min(0).values > gap


def _backend(name, dtype, max_batch=8, ctx=512, kv_tokens=2048):
    from inference_b200.engine.loading import gpu_backend
    from inference_b200.models import ModelConfig

    cfg, w, _ = _model(name)
    return gpu_backend(ModelConfig.from_json(cfg), w, dtype=dtype, max_batch=max_batch, max_context=ctx, kv_tokens=kv_tokens)


def _feed(backend, seq, tokens, cuts):
    """Feeds `tokens` in portions of the given sizes (the last size repeats); logits of every position."""
    out, at = [], 0
    while at < len(tokens):
        n = min(cuts.pop(0) if len(cuts) > 1 else cuts[0], len(tokens) - at)
        out.append(backend.forward_at([seq], [tokens[at:at + n]], [list(range(n))]).clone())
        at += n
    return torch.cat(out)


def _idle(backend):
    return backend.runner.pool.allocator.live_blocks() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ref.MODELS))
def test_every_layer_matches(name, dtype):
    from inference_b200.engine.kv_pool import PagedSequence

    b = _backend(name, dtype)
    model, tokens, got = b.runner.model, _tokens(name, 60, 1), []
    fwd = model.forward_hidden
    model.forward_hidden = lambda inp, kv: fwd(inp, kv, tap=got.append)
    b.runner.prefill([PagedSequence(b.runner.pool)], [tokens], want=[[0]])
    trail = _want(name, tokens)[1]
    assert len(got) == len(trail)
    for i, (x, y) in enumerate(zip(got, trail)):
        assert rel(x, y) < TOL[dtype], (i, rel(x, y))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ref.MODELS))
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [3, 2, 7, 16, 17, 31], [64], [100, 1]])
def test_prompts_portions_and_decoding_agree(name, dtype, cuts):
    """Whole prompt, token by token (graph-replayed decode), and portions from two tokens up give the same logits."""
    tokens = _tokens(name, 139, 2)
    b = _backend(name, dtype)
    got = _feed(b, b.new_sequence(), tokens, list(cuts))
    want = _want(name, tokens)[0]
    assert rel(got, want) < TOL[dtype]
    sure = _sure(name, tokens)
    assert int(sure.sum()) > 60
    worst = max(rel(g, w) for g, w, ok in zip(got, want, sure) if ok or dtype == torch.float32)
    assert worst < 4 * TOL[dtype], worst


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_contexts_decode_with_split_kv(dtype):
    tokens = _tokens("d", 700, 3)
    want = _want("d", tokens)[0]
    b = _backend("d", dtype, ctx=800, kv_tokens=704)
    seq = b.new_sequence()
    got = _feed(b, seq, tokens, [480, 50, 5, 12, 1])
    assert rel(got, want) < TOL[dtype] and rel(got[-150:], want[-150:]) < TOL[dtype]
    assert max(b.runner.model.decode_splits(1, 700)) > 1


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_and_reused_pages(dtype):
    """Portions of some sequences beside single tokens of others, sequences that pause, end and give their pages to new ones; the pages
    are just enough. Every logit equals that of the sequence alone."""
    lens = {"p": 90, "q": 33, "r": 150, "s": 17, "t": 120, "u": 64}
    toks = {k: _tokens("a", n, 10 + i) for i, (k, n) in enumerate(lens.items())}
    b = _backend("a", dtype, max_batch=4, ctx=160, kv_tokens=352)
    steps = [{"p": 40, "q": 2, "r": 5}, {"p": 1, "q": 1, "r": 60, "s": 16}, {"q": 30, "s": 1}, {"p": 1, "r": 1}, {"p": 2, "r": 37},
             {"p": 46, "r": 2, "t": 100}, {"r": 45, "t": 1}, {"t": 1, "u": 1}, {"t": 2, "u": 3}, {"t": 1, "u": 1}, {"u": 57, "t": 15},
             {"u": 1}, {"u": 1}]
    seqs, at, got = {}, {k: 0 for k in lens}, {k: [] for k in lens}
    for step in steps:
        for k in step:
            if k not in seqs:
                seqs[k] = b.new_sequence()
        out = b.forward_at([seqs[k] for k in step], [toks[k][at[k]:at[k] + n] for k, n in step.items()],
                           [list(range(n)) for n in step.values()]).clone()
        o = 0
        for k, n in step.items():
            got[k].append(out[o:o + n])
            o, at[k] = o + n, at[k] + n
            if at[k] == lens[k]:
                b.release(seqs.pop(k))
    assert not seqs and _idle(b)
    for k in lens:
        assert rel(torch.cat(got[k]), _want("a", toks[k])[0]) < TOL[dtype], k


def test_wanted_places_only():
    b, tokens = _backend("b", torch.float32), _tokens("b", 30, 4)
    want = _want("b", tokens)[0]
    s, t = b.new_sequence(), b.new_sequence()
    assert b.forward_at([s], [tokens[:10]], [[]]) is None
    got = b.forward_at([s, t], [tokens[10:20], tokens[:4]], [[9, 0], [2]])
    assert rel(got, want[[19, 10, 2]]) < TOL[torch.float32]
    assert rel(b.forward_at([s, t], [[tokens[20]], [tokens[4]]], [[], [0]]), want[[4]]) < TOL[torch.float32]


def _check_greedy(name, prompt, got, steps, slack):
    logits = _want(name, prompt + got)[0]
    for i in range(steps):      # teacher-forced on what was generated: each token is the best one, or tied within rounding
        row = logits[len(prompt) - 1 + i]
        assert float(row.max() - row[got[i]]) <= slack * float(row.std()), (i, got[i], int(row.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "b"])
def test_greedy_generation_loops(name, dtype):
    from inference_b200.engine.decode import (ContinuousConfig, ContinuousRequest, GenerationConfig, PrefixCache, generate,
                                              generate_batch, generate_cached, generate_continuous, generate_draft_speculative,
                                              generate_prompt_lookup)
    from inference_b200.engine.llm_engine import EngineConfig, LlmEngine
    from inference_b200.engine.loading import gpu_backend
    from inference_b200.models import ModelConfig

    slack = 1e-4 if dtype == torch.float32 else 0.15
    mcfg, w, _ = _model(name)
    b = gpu_backend(ModelConfig.from_json(mcfg), w, dtype=dtype, max_batch=8, max_context=512)
    prompts = [_tokens(name, n, 20 + n) for n in (35, 2, 70, 19, 50)]
    cfg = GenerationConfig(max_new_tokens=12)
    runs = [[generate(b, p, cfg).tokens for p in prompts], [r.tokens for r in generate_batch(b, prompts, cfg)]]
    for chunk in (0, 16):
        reqs = [ContinuousRequest(p, 12) for p in prompts]
        runs.append([r.tokens for r in generate_continuous(b, reqs, ContinuousConfig(max_batch=3, prefill_chunk=chunk))])
    cache = PrefixCache(b, capacity=8)
    runs.append([generate_cached(b, cache, p, cfg).tokens for p in prompts])
    more = [p + _tokens(name, 9, 3) for p in prompts]
    longer = [generate_cached(b, cache, p, cfg).tokens for p in more]              # continues the cached prompts
    assert cache.stats.hits > 0
    for p, t in zip(more, longer):
        _check_greedy(name, p, t, 12, slack)
    cache.clear()
    runs.append([generate_prompt_lookup(b, p, cfg)[0].tokens for p in prompts])    # rolls rejected drafts back
    draft = gpu_backend(ModelConfig.from_json(mcfg), ref.random_weights(mcfg, seed=5), dtype=dtype, max_batch=2, max_context=512)
    runs.append([generate_draft_speculative(b, draft, p, cfg)[0].tokens for p in prompts])
    eng = LlmEngine(b.runner.model, EngineConfig(max_batch=8, max_seq_len=256))
    runs.append(eng.generate_batch(prompts, 12).tokens)
    seqs = [eng.new_sequence() for _ in prompts]
    first = eng.prefill_batch(seqs, prompts)
    multi = eng.runner.decode_multi(seqs, first, 11).t().tolist()                   # tokens fed back on the device
    runs.append([[f] + m for f, m in zip(first, multi)])
    assert _idle(b) and _idle(draft)
    for tokens in runs:
        for p, t in zip(prompts, tokens):
            assert len(t) == 12
            _check_greedy(name, p, t, 12, slack)
    if dtype == torch.float32:
        assert all(r == runs[0] for r in runs[1:])


def test_greedy_tokens_equal_the_restatement():
    from inference_b200.engine.decode import GenerationConfig, generate

    cfg, w, _ = _model("b")
    prompt = _tokens("b", 20, 5)
    want, gaps = ref.greedy(cfg, w, prompt, 10)
    assert generate(_backend("b", torch.float32), prompt, GenerationConfig(max_new_tokens=10)).tokens == want, gaps


@pytest.mark.parametrize("dtype", DTYPES)
def test_large_batches_pad_to_a_bucket(dtype):
    """19 rows decode in a graph captured for 24; the padding rows change nothing."""
    b = _backend("b", dtype, max_batch=24, ctx=64, kv_tokens=24 * 64)
    toks = [_tokens("b", 12 + i, 100 + i) for i in range(19)]
    seqs = [b.new_sequence() for _ in toks]
    b.forward_at(seqs, [t[:-3] for t in toks], [[] for _ in toks])
    for back in (3, 2, 1):
        got = b.forward_at(seqs, [[t[-back]] for t in toks], [[0] for _ in toks])
        for g, t in zip(got, toks):
            if dtype == torch.float32 or _sure("b", t)[-back]:
                assert rel(g, _want("b", t)[0][-back]) < (TOL[dtype] if dtype == torch.float32 else 4 * TOL[dtype])


# ---- provider and replay tool ------------------------------------------------------------------------------------------
def _snapshot(path: Path, name: str, tokenizer=False) -> Path:
    from inference_b200.io.safetensors_io import save_file
    from inference_b200.testkit.synthetic import wordlevel_tokenizer_json

    cfg, w, _ = _model(name)
    path.mkdir(parents=True, exist_ok=True)
    save_file(w, path / "model.safetensors")
    (path / "config.json").write_text(json.dumps(cfg))
    if tokenizer:
        (path / "tokenizer.json").write_text(wordlevel_tokenizer_json(cfg["vocab"]))
        (path / "tokenizer_config.json").write_text("{}")
    return path


def test_catalog_provider_generates(tmp_path):
    from inference_b200.bundles import runtime_b200
    from inference_b200.contracts.core_llm import LoadSpec, Message, Sampling, TextLlmRequest

    llm = runtime_b200.catalog().text().load_for_model(LoadSpec.dense(str(_snapshot(tmp_path / "m", "a", tokenizer=True))))
    assert llm.descriptor().family == "rotalorn"
    req = TextLlmRequest(messages=[Message.user("hello world the cat")], max_new_tokens=8, sampling=Sampling(temperature=0.0))
    events = []
    out = llm.generate(req, events.append)
    assert 0 < out.usage.generated_tokens <= 8 and events
    hot = TextLlmRequest(messages=[Message.user("hello world the cat")], max_new_tokens=8, seed=3,
                         sampling=Sampling(temperature=0.9, top_p=0.9))
    assert llm.generate(hot, lambda e: None).text == llm.generate(hot, lambda e: None).text


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_replays_steps(tmp_path, dtype):
    d, out = _snapshot(tmp_path / "m", "a"), tmp_path / "out"
    x, y = _tokens("a", 80, 6), _tokens("a", 45, 7)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": x[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": x[50:51], "want": [0]}, {"id": "y", "tokens": y, "want": [44]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": x[51:52], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "x", "tokens": x[52:], "want": [27, 1]}], "end": ["x"]}]
    r = subprocess.run([sys.executable, str(Path(__file__).resolve().parent.parent / "bin" / "trace_run"), "--model", str(d),
                        "--dtype", dtype, "--out", str(out), "--max-tokens", "144"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    wx, wy = _want("a", x)[0], _want("a", y)[0]
    want = {0: wx[[0, 49]], 1: torch.stack([wx[50], wy[44]]), 3: wx[[79, 53]]}
    assert sorted(p.name for p in out.iterdir()) == [f"{i}.f32" for i in want]
    for i, w in want.items():
        got = torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(len(w), -1)
        assert rel(got, w) < TOL[getattr(torch, dtype)]
