"""Zobunex on the GPU against the plain float64 restatement in tests/zobunex_reference.py: each mechanism alone, then whole
models in float32 and bfloat16 through the runner, the paged pool, the generation loops, the provider and the replay tool."""
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import zobunex_reference as ref

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


# ---- mechanisms alone -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,Hp", [(160, 160), (90, 96), (1, 8), (512, 512), (1030, 1032), (1024, 1024), (2048, 2048), (4096, 4096),
                                  (8192, 8192), (9000, 9000), (16384, 16384)])
@pytest.mark.parametrize("center", [True, False])
def test_stream_norm_joins_norms_and_writes(H, Hp, center):
    from inference_b200 import ops

    T, eps = 5, 1e-2
    pad = lambda t: torch.nn.functional.pad(t, (0, Hp - H)).cuda().contiguous()   # noqa: E731
    x, y = rnd(T, H, seed=1) + 3.0, rnd(T, H, seed=2) * 2 + 1.0
    w1, b1, w2, b2 = (rnd(H, seed=s) for s in (3, 4, 5, 6))
    n = (lambda t, w, b: ref.layer_norm(t, w, b, eps)) if center else (lambda t, w, b: ref.rms_norm(t, w, eps))
    d = [t.double() for t in (x, y, w1, b1, w2, b2)]
    xs = d[0] + n(d[1], d[2], d[3])
    want = n(xs, d[4], d[5]) * 0.7
    n1 = ops.NormWeights(pad(w1), pad(b1) if center else None)
    n2 = ops.NormWeights(pad(w2), pad(b2) if center else None)
    gx, out = pad(x), torch.full((T, Hp), 9.0, device="cuda")
    ops.stream_norm(gx, H, eps, branch=ops.Branch(pad(y), n1), norm=n2, out=out, center=center, out_scale=0.7)
    assert rel(gx[:, :H], xs) < 1e-6 and rel(out[:, :H], want) < 2e-6
    assert (gx[:, H:] == 0).all() and (out[:, H:] == 0).all()
    # bf16 branch and output
    yb = y.to(torch.bfloat16)
    gx, out = pad(x), torch.empty((T, Hp), device="cuda", dtype=torch.bfloat16)
    ops.stream_norm(gx, H, eps, branch=ops.Branch(pad(yb), n1), norm=n2, out=out, center=center)
    xs = d[0] + n(yb.double(), d[2], d[3])
    assert rel(gx[:, :H], xs) < 1e-6 and rel(out[:, :H], n(xs, d[4], d[5])) < 4e-3
    # chosen rows of the stream, no branch
    rows = torch.tensor([3, 0], device="cuda")
    out = torch.empty((2, Hp), device="cuda")
    ops.stream_norm(pad(x), H, eps, norm=n2, out=out, rows=rows, center=center)
    assert rel(out[:, :H], n(d[0], d[4], d[5])[[3, 0]]) < 2e-6


def test_stream_norm_gathers_the_branch_and_scatters_the_rows():
    from inference_b200 import ops

    T, H, top, R = 4, 40, 3, 20
    x, y = rnd(T, H, seed=1), rnd(R, H, seed=2)
    dest = torch.randperm(R, generator=torch.Generator().manual_seed(0))[:T * top].view(T, top)
    w, b = rnd(H, seed=3), rnd(H, seed=4)
    xs = x.double() + ref.layer_norm(y.double()[dest].sum(1) / top, w.double(), b.double(), 1e-5)
    gx, out = x.cuda(), torch.zeros((R, H), device="cuda")
    d = dest.int().cuda()
    nw = ops.NormWeights(w.cuda(), b.cuda())
    ops.stream_norm(gx, H, 1e-5, branch=ops.Branch(y.cuda(), nw, d, top, 1.0 / top), norm=nw, out=out, out_rows=d, out_top=top)
    assert rel(gx, xs) < 1e-6
    want = torch.zeros(R, H, dtype=F)
    want[dest.reshape(-1)] = ref.layer_norm(xs, w.double(), b.double(), 1e-5).repeat_interleave(top, 0)
    assert rel(out, want) < 2e-6
    # without a norm the stream itself is stored
    out = torch.empty((T, H), device="cuda")
    ops.stream_norm(gx, H, 1e-5, out=out)
    assert torch.equal(out, gx)


@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_embed_copies_rows(dtype):
    from inference_b200 import ops

    table = rnd(30, 24, dtype=dtype).cuda()
    ids = torch.tensor([4, 29, 0, 4], device="cuda")
    cat = torch.zeros((4, 48), dtype=dtype, device="cuda")
    x = ops.stream_embed(ids, table, copies=[cat[:, 24:], cat[:, :24]])
    assert torch.equal(x, table.float()[ids]) and torch.equal(cat, torch.cat([table[ids], table[ids]], 1))


@pytest.mark.parametrize("T,E,top", [(1, 5, 3), (7, 16, 1), (300, 3, 2), (2500, 40, 4), (64, 1, 1)])
@pytest.mark.parametrize("padded", [False, True])
def test_table_routing_lays_pairs_out_by_expert(T, E, top, padded):
    from inference_b200 import ops

    L, V = 3, 50
    g = torch.Generator().manual_seed(T)
    tables = torch.stack([torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(V)]) for _ in range(L)]).int()
    ids = torch.randint(0, V, (T,), generator=g)
    for lay, plan in enumerate(ops.table_routing(ids.cuda(), tables.cuda(), E, padded=padded)):
        dest, off = plan.dest.cpu().long(), plan.offsets.cpu()
        want = tables[lay].long()[ids]
        flat = dest.reshape(-1)
        assert flat.unique().numel() == T * top and flat.min() >= 0 and flat.max() < plan.rows
        assert ((off[want] <= dest) & (dest < off[want + 1])).all()
        if padded:
            assert (off % 128 == 0).all()
            tg = plan.tile_group.cpu().long()
            assert torch.equal(tg[dest // 128], want) and (tg[off[-1] // 128:] == -1).all()
        else:
            assert off[-1] == T * top
            assert torch.equal(plan.src.cpu().long()[flat].view(T, top), torch.arange(T)[:, None].expand(T, top))
            act = plan.active.cpu()
            assert sorted(act[act >= 0].tolist()) == sorted(set(want.reshape(-1).tolist()))


@pytest.mark.parametrize("dtype,padded", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
@pytest.mark.parametrize("T,H,ff,E,top", [(1, 64, 24, 7, 2), (9, 200, 56, 5, 3), (130, 328, 136, 3, 1), (600, 96, 40, 4, 4)])
def test_routed_experts(dtype, padded, T, H, ff, E, top):
    from inference_b200 import ops

    V = 31
    g = torch.Generator().manual_seed(T)
    table = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(V)])
    ids = torch.randint(0, V, (T,), generator=g)
    x, up, down = (rnd(*s, seed=i, dtype=torch.bfloat16, std=sd).to(dtype) for i, (s, sd) in enumerate(
        [((T, H), 1.0), ((E, ff, H), H ** -0.5), ((E, H, ff), ff ** -0.5)]))
    plan = ops.table_routing(ids.cuda(), table.int()[None].cuda(), E, padded=padded)[0]
    h = x.cuda()
    if padded:
        h = torch.zeros((plan.rows, H), dtype=dtype, device="cuda")
        h[plan.dest.long().reshape(-1)] = x.cuda().repeat_interleave(top, 0)
    y = ops.routed_ffn(h, up.cuda(), down.cuda(), plan, "relu2")
    got = y[plan.dest.long().reshape(-1)].view(T, top, H).double().mean(1)
    want = ref.table_experts(x.double(), ids, table, up.double(), down.double())
    assert rel(got, want) < OP_TOL[dtype]


@pytest.mark.parametrize("T,N,K", [(1, 3, 5), (70, 130, 33), (200, 64, 512)])
def test_gemm_f32_is_true_32_bit(T, N, K):
    from inference_b200 import ops

    a, w = rnd(T, K, seed=1), rnd(N, K, seed=2)
    assert rel(ops.gemm_f32(a.cuda(), w.cuda()), a.double() @ w.double().T) < 1e-6
    want = torch.relu(a.double() @ w.double().T).square()
    assert rel(ops.gemm_f32(a.cuda(), w.cuda(), act="relu2"), want) < 2e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,Dv,rot", [(64, 32, 24), (40, 72, 40), (128, 128, 128), (160, 136, 2), (16, 300, 0)])
def test_rotation_and_paged_write(dtype, D, Dv, rot):
    from inference_b200 import ops

    T, Hq, Hkv, bs, nblk = 6, 4, 2, 16, 5
    qkv = rnd(T, (Hq + Hkv) * D + Hkv * Dv, dtype=dtype)
    pos = torch.tensor([0, 1, 7, 40, 2, 63])
    slots = torch.tensor([70, 3, 16, 15, -1, 33])
    ang = torch.arange(64, dtype=F)[:, None] * 300.0 ** (-2.0 * torch.arange(rot // 2, dtype=F) / max(rot, 1))
    kc, vc = (torch.zeros((nblk, Hkv, bs, d), dtype=dtype, device="cuda") for d in (D, Dv))
    buf = qkv.cuda()
    ops.rope_kv_write(buf, pos.int().cuda(), slots.cuda(), ang.cos().float().cuda(), ang.sin().float().cuda(), kc, vc, Hq, Hkv, D,
                      rot_dim=rot, interleaved=True, block_size=bs, v_dim=Dv)
    q, k, v = qkv.double().split([Hq * D, Hkv * D, Hkv * Dv], 1)
    q, k = (ref.rotate_pairs(t.view(T, -1, D), pos, rot, 300.0) for t in (q, k))
    assert rel(buf[:, :Hq * D].view(T, Hq, D), q) < OP_TOL[dtype]
    assert rel(buf[:4, Hq * D:(Hq + Hkv) * D].view(4, Hkv, D), k[:4]) < OP_TOL[dtype]
    for t in (0, 1, 2, 3, 5):
        b, o = divmod(int(slots[t]), bs)
        assert rel(kc[b, :, o], k[t]) < OP_TOL[dtype] and torch.equal(vc[b, :, o].cpu().double(), v[t].view(Hkv, Dv))
    assert int((vc != 0).any(-1).sum()) == 5 * Hkv         # the token without a slot wrote nothing


def _paged(k, v, lens, dtype, bs=16, seed=0):
    """Scatters each sequence's keys / values over shuffled pages; unused page rows hold large values."""
    G = k[0].shape[1]
    need = [(n + bs - 1) // bs for n in lens]
    perm = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    kc, vc = (torch.full((len(perm), G, bs, t[0].shape[2]), 7.0, dtype=dtype) for t in (k, v))
    table = torch.zeros((len(lens), max(need) + 2), dtype=torch.int32)
    for s, n in enumerate(lens):
        for b in range(need[s]):
            page = perm.pop()
            table[s, b] = page
            m = min(bs, n - b * bs)
            kc[page, :, :m] = k[s][b * bs:b * bs + m].transpose(0, 1).to(dtype)
            vc[page, :, :m] = v[s][b * bs:b * bs + m].transpose(0, 1).to(dtype)
    return kc.cuda(), vc.cuda(), table.cuda()


def _attention_case(dtype, H, G, D, Dv, chunk, lens, q_lens, mode, splits=1, scale=None, kernel="auto", sink_mean=0.0, plant=None):
    """Random keys, plus planted ones: the last query of every sequence is aligned with one key (`plant` positions before its
    chunk's start when negative, after it otherwise), so that a wrong edge moves nearly all of its weight."""
    from inference_b200 import ops

    scale = D ** -0.5 if scale is None else scale
    ks = [rnd(n, G, D, seed=10 + i, dtype=torch.bfloat16).float() for i, n in enumerate(lens)]
    vs = [rnd(n, G, Dv, seed=30 + i, dtype=torch.bfloat16).float() for i, n in enumerate(lens)]
    qs = [rnd(n, H, D, seed=50 + i, dtype=torch.bfloat16).float() for i, n in enumerate(q_lens)]
    if plant is not None:
        for k, q, n in zip(ks, qs, lens):
            at = (n - 1) // chunk * chunk + plant if chunk else plant
            if 0 <= at < n:
                u = torch.nn.functional.normalize(rnd(D, seed=99), dim=0)
                k[at], q[-1] = (u * 8).bfloat16().float(), (u * 12.0 / (8 * scale)).bfloat16().float()
    sink = rnd(H, seed=7) + sink_mean
    want = torch.cat([ref.attention(q.double(), k.double(), v.double(), torch.arange(n - len(q), n), scale, chunk, sink.double())
                      for q, k, v, n in zip(qs, ks, vs, lens)])
    kc, vc, table = _paged(ks, vs, lens, dtype)
    q = torch.cat(qs).to(dtype).cuda()
    cu = torch.tensor([0] + q_lens).cumsum(0).int().cuda()
    fresh = None
    if mode == "fresh":
        buf = torch.cat([torch.cat(t).reshape(sum(lens), -1) for t in (qs, ks, vs)], 1).to(dtype).cuda()
        q = buf[:, :H * D].view(-1, H, D)
        fresh = (buf[:, H * D:(H + G) * D].view(-1, G, D), buf[:, (H + G) * D:].view(-1, G, Dv))
    got = ops.chunk_attention(q, kc, vc, table, torch.tensor(lens).int().cuda(), cu_q=None if mode == "decode" else cu,
                              max_q_len=max(q_lens), scale=scale, chunk=chunk, sink=sink.cuda(), decode=mode == "decode",
                              num_splits=splits, fresh_kv=fresh, kernel=kernel)
    ops.check_status()
    return rel(got.view(-1, H, Dv), want)


SHAPES = [(4, 2, 64, 64), (6, 3, 64, 32), (4, 1, 40, 72), (2, 2, 128, 128), (8, 2, 16, 24), (3, 3, 128, 8), (8, 1, 104, 120)]


@pytest.mark.parametrize("H,G,D,Dv", SHAPES)
@pytest.mark.parametrize("mode", ["fresh", "paged"])
@pytest.mark.parametrize("chunk", [0, 1, 16, 37, 128, 300])
def test_chunk_attention_prefill(H, G, D, Dv, mode, chunk):
    lens = [401, 1, 130, 257, 37]
    q_lens = lens if mode == "fresh" else [150, 1, 2, 257, 20]
    assert _attention_case(torch.bfloat16, H, G, D, Dv, chunk, lens, q_lens, mode) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("chunk", [16, 37, 90, 128, 300])
@pytest.mark.parametrize("plant", [-17, -1, 0, 1])
@pytest.mark.parametrize("mode", ["fresh", "paged", "decode"])
def test_chunk_edges_carry_the_weight(chunk, plant, mode):
    """A key that would take the whole softmax sits just inside / outside the last query's chunk."""
    for last in (0, 1, chunk - 1):
        n = 2 * chunk + last + 1
        lens = [n, n + chunk]
        q_lens = lens if mode == "fresh" else [1, 1] if mode == "decode" else [2, 3]
        for dtype in DTYPES if mode != "fresh" else DTYPES[1:]:
            err = _attention_case(dtype, 4, 2, 64, 48, chunk, lens, q_lens, mode, plant=plant)
            assert err < OP_TOL[dtype], (last, dtype, err)


@pytest.mark.parametrize("H,G,D,Dv", SHAPES)
@pytest.mark.parametrize("chunk,splits", [(0, 1), (0, 4), (0, 16), (37, 1), (300, 2), (300, 8), (1000, 16)])
def test_chunk_attention_decode(H, G, D, Dv, chunk, splits):
    lens = [1, 16, 17, 300, 301, 640, 1023]
    assert _attention_case(torch.bfloat16, H, G, D, Dv, chunk, lens, [1] * 7, "decode", splits) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("chunk", [0, 37, 64])
def test_chunk_attention_decodes_several_tokens_per_sequence(chunk):
    for lens in ([38, 75, 130], [40, 66, 200]):
        assert _attention_case(torch.bfloat16, 4, 2, 64, 32, chunk, lens, [4] * 3, "decode", 2) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv,scale", [(2, 1, 160, 136, None), (34, 2, 24, 24, None), (4, 2, 33, 7, None), (4, 2, 64, 64, -0.2)])
def test_chunk_attention_outside_the_tensor_core_kernels(dtype, H, G, D, Dv, scale):
    for chunk in (0, 37):
        assert _attention_case(dtype, H, G, D, Dv, chunk, [100, 3, 75], [100, 2, 40], "paged", scale=scale) < OP_TOL[dtype]
        assert _attention_case(dtype, H, G, D, Dv, chunk, [100, 3, 75], [1] * 3, "decode", scale=scale) < OP_TOL[dtype]


@pytest.mark.parametrize("mean", [-40.0, 6.0, 60.0])
@pytest.mark.parametrize("mode,splits", [("fresh", 1), ("paged", 1), ("decode", 1), ("decode", 4)])
def test_sinks_of_any_size(mean, mode, splits):
    """A sink far below the scores changes nothing, one far above them silences the head."""
    lens = [200, 130]
    q_lens = [1, 1] if mode == "decode" else lens if mode == "fresh" else [50, 2]
    assert _attention_case(torch.bfloat16, 4, 2, 64, 64, 90, lens, q_lens, mode, splits, sink_mean=mean) < OP_TOL[torch.bfloat16]


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


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_every_layer_run_matches(name, dtype):
    from inference_b200.engine.kv_pool import PagedSequence

    b = _backend(name, dtype)
    model, tokens, got = b.runner.model, _tokens(name, 60, 1), []
    fwd = model.forward_hidden
    model.forward_hidden = lambda inp, kv: fwd(inp, kv, tap=got.append)
    b.runner.prefill([PagedSequence(b.runner.pool)], [tokens], want=[[0]])
    logits, trail = _want(name, tokens)
    assert len(got) == len(trail) == len(ref.schedule(_model(name)[0]))
    for r, (x, y) in enumerate(zip(got, trail)):
        assert rel(x, y) < TOL[dtype], (r, rel(x, y))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "b", "c"])
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [3, 2, 7, 16, 17, 31], [64], [100, 1]])
def test_prompts_portions_and_decoding_agree(name, dtype, cuts):
    """Whole prompt, token by token (graph-replayed decode), and portions from two tokens up give the same logits."""
    tokens = _tokens(name, 139, 2)
    b = _backend(name, dtype)
    got = _feed(b, b.new_sequence(), tokens, list(cuts))
    want = _want(name, tokens)[0]
    assert rel(got, want) < TOL[dtype]
    worst = max(rel(g, w) for g, w in zip(got, want))
    assert worst < 4 * TOL[dtype], worst


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_context_decodes_across_chunks_with_split_kv(dtype):
    """1024 tokens: the last portion starts inside a chunk, decoding then passes the edges of both layers' chunks."""
    tokens = _tokens("d", 1024, 3)
    want = _want("d", tokens)[0]
    b = _backend("d", dtype, ctx=1100, kv_tokens=1104)
    seq = b.new_sequence()
    got = _feed(b, seq, tokens, [640, 50, 1])
    assert rel(got, want) < TOL[dtype]
    for lo, hi in ((690, 720), (990, 1024)):
        assert rel(got[lo:hi], want[lo:hi]) < TOL[dtype]
    assert max(b.runner.model.decode_splits(1, 1000)) > 1


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_and_reused_pages(dtype):
    """Portions of some sequences beside single tokens of others, sequences that pause, end and give their pages to new
    ones; the pool is just large enough. Every logit equals that of the sequence alone."""
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
    assert not seqs and b.runner.pool.allocator.live_blocks() == 0
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
    cfg, w, _ = _model(name)
    logits = _want(name, prompt + got)[0]
    for i in range(steps):      # teacher-forced on what was generated: each token is the best one, or tied within rounding
        row = logits[len(prompt) - 1 + i]
        assert float(row.max() - row[got[i]]) <= slack * float(row.std()), (i, got[i], int(row.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_loops(dtype):
    from inference_b200.engine.decode import (ContinuousConfig, ContinuousRequest, GenerationConfig, PrefixCache, generate,
                                              generate_batch, generate_cached, generate_continuous, generate_prompt_lookup)
    from inference_b200.engine.llm_engine import EngineConfig, LlmEngine

    slack = 1e-4 if dtype == torch.float32 else 0.15
    b = _backend("a", dtype)
    prompts = [_tokens("a", n, 20 + n) for n in (35, 2, 70, 19, 50)]
    cfg = GenerationConfig(max_new_tokens=12)
    runs = [[generate(b, p, cfg).tokens for p in prompts], [r.tokens for r in generate_batch(b, prompts, cfg)]]
    for chunk in (0, 16):
        reqs = [ContinuousRequest(p, 12) for p in prompts]
        runs.append([r.tokens for r in generate_continuous(b, reqs, ContinuousConfig(max_batch=3, prefill_chunk=chunk))])
    cache = PrefixCache(b, capacity=8)
    runs.append([generate_cached(b, cache, p, cfg).tokens for p in prompts])
    runs.append([generate_cached(b, cache, p, cfg).tokens for p in prompts])       # every prompt again, from cached pages
    assert cache.stats.hits > 0
    cache.clear()
    runs.append([generate_prompt_lookup(b, p, cfg)[0].tokens for p in prompts])    # rolls rejected drafts back
    eng = LlmEngine(b.runner.model, EngineConfig(max_batch=8, max_seq_len=256))
    runs.append(eng.generate_batch(prompts, 12).tokens)
    seqs = [eng.new_sequence() for _ in prompts]
    first = eng.prefill_batch(seqs, prompts)
    multi = eng.runner.decode_multi(seqs, first, 11).t().tolist()                   # tokens fed back on the device
    runs.append([[f] + m for f, m in zip(first, multi)])
    assert b.runner.pool.allocator.live_blocks() == 0
    for tokens in runs:
        for p, t in zip(prompts, tokens):
            assert len(t) == 12
            _check_greedy("a", p, t, 12, slack)
    if dtype == torch.float32:
        assert all(r == runs[0] for r in runs[1:])


def test_greedy_tokens_equal_the_restatement():
    from inference_b200.engine.decode import GenerationConfig, generate

    cfg, w, _ = _model("b")
    prompt = _tokens("b", 20, 5)
    want, gaps = ref.greedy(cfg, w, prompt, 10)
    assert generate(_backend("b", torch.float32), prompt, GenerationConfig(max_new_tokens=10)).tokens == want, gaps


def test_large_batches_pad_to_a_bucket():
    b = _backend("b", torch.bfloat16, max_batch=24, ctx=64, kv_tokens=24 * 64)
    toks = [_tokens("b", 12 + i, 100 + i) for i in range(19)]
    seqs = [b.new_sequence() for _ in toks]
    b.forward_at(seqs, [t[:-2] for t in toks], [[] for _ in toks])
    for back in (2, 1):
        got = b.forward_at(seqs, [[t[-back]] for t in toks], [[0] for _ in toks])
        for g, t in zip(got, toks):
            assert rel(g, _want("b", t)[0][-back]) < 4 * TOL[torch.bfloat16]


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
    assert llm.descriptor().family == "zobunex"
    req = TextLlmRequest(messages=[Message.user("hello world the cat")], max_new_tokens=8,
                         sampling=Sampling(temperature=0.0))
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
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    wx, wy = _want("a", x)[0], _want("a", y)[0]
    want = {0: wx[[0, 49]], 1: torch.stack([wx[50], wy[44]]), 3: wx[[79, 53]]}
    assert sorted(p.name for p in out.iterdir()) == [f"{i}.f32" for i in want]
    for i, w in want.items():
        got = torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(len(w), -1)
        assert rel(got, w) < TOL[getattr(torch, dtype)]
