"""Nafelix on the GPU against the plain float64 restatement in tests/nafelix_reference.py: each mechanism alone, then whole models in
float32 and bfloat16 through the runner, the paged pool, the generation loops, the provider and the replay tool."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import nafelix_reference as ref

pytestmark = pytest.mark.gpu
F = torch.float64
DTYPES = [torch.float32, torch.bfloat16]
# relative RMS error of logits / of one mechanism's output
TOL = {torch.float32: 2e-5, torch.bfloat16: 4e-2}
OP_TOL = {torch.float32: 1e-5, torch.bfloat16: 8e-3}


def rel(got, want):
    got, want = got.detach().double().cpu(), want.double().cpu()
    return float((got - want).square().mean().sqrt() / want.square().mean().sqrt().clamp_min(1e-12))


def rnd(*shape, seed=0, dtype=torch.float32, std=1.0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * std).to(dtype)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def up8(n):
    return (n + 7) // 8 * 8


# ---- streams -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,H,Hp", [(1, 90, 96), (2, 144, 144), (3, 264, 264), (4, 1030, 1032), (5, 600, 600), (8, 2048, 2048), (3, 4096, 4096),
                                    (16, 520, 520), (2, 8200, 8200), (4, 3000, 3000)])
def test_streams_are_read_and_joined(dtype, S, H, Hp):
    """Plain, doubly normed and routed branches; all streams alike at first; in place; chosen rows."""
    from inference_b200 import ops

    T, eps, R = 5, 1e-2, 23
    pad = lambda t: torch.nn.functional.pad(t, (0, Hp - H)).cuda().contiguous()   # noqa: E731
    nw = lambda t: ops.NormWeights(pad(t))                                          # noqa: E731
    x0, y, y2, e = rnd(T, H, seed=1) + 2, *(rnd(n, H, seed=s, dtype=dtype) for n, s in ((T, 2), (T, 3), (R, 4)))
    w, w1, w2 = rnd(H, seed=5), rnd(H, seed=6), rnd(H, seed=7)
    mix, put, read = rnd(S, S, seed=8), rnd(S, seed=9), rnd(S, seed=10)
    rows = torch.stack([torch.randperm(R, generator=torch.Generator().manual_seed(t))[:3] for t in range(T)])
    share = rnd(T, 3, seed=11).abs()
    join = ops.StreamMix(mix.cuda(), put.cuda())
    tol = {torch.float32: 3e-6, torch.bfloat16: 4e-3}[dtype]
    # nothing to join: the first sublayer's input
    out = torch.full((T, Hp), 9.0, dtype=dtype, device="cuda")
    ops.hyper_step(pad(x0), S, H, eps, read=read.cuda(), norm=nw(w), out=out)
    xs = x0.double()[None].expand(S, -1, -1)
    assert rel(out[:, :H], ref.rms(ref.read_streams(xs, read.double()), eps) * w.double()) < tol and (out[:, H:] == 0).all()
    # from the common row into the streams, then in place
    streams = torch.full((T, S, Hp), 7.0, device="cuda")
    half = lambda t: (t.double() * 0.5).float()   # noqa: E731
    kinds = [(ops.HyperBranch(pad(y)), y.double()),
             (ops.HyperBranch(pad(y), nw(half(w1)), pad(y2), nw(half(w2))),
              0.5 * (ref.rms(y.double(), eps) * w1.double() + ref.rms(y2.double(), eps) * w2.double())),
             (ops.HyperBranch(ops.RoutedRows(pad(e), rows.int().cuda(), share.cuda())), (e.double()[rows] * share.double()[..., None]).sum(1)),
             (ops.HyperBranch(pad(y2), nw(w1)), ref.rms(y2.double(), eps) * w1.double())]
    src = pad(x0)
    for branch, plain in kinds:
        xs = ref.write_streams(xs, mix.double(), put.double(), plain)
        ops.hyper_step(src, S, H, eps, branch=branch, join=join, x_out=streams, read=read.cuda(), norm=nw(w), out=out)
        src = streams
        assert rel(streams[..., :H].transpose(0, 1), xs) < 3e-6 and (streams[..., H:] == 0).all()
        assert rel(out[:, :H], ref.rms(ref.read_streams(xs, read.double()), eps) * w.double()) < tol and (out[:, H:] == 0).all()
    # joined without reading; the sum of the streams of chosen rows
    xs = ref.write_streams(xs, mix.double(), put.double(), y.double())
    assert ops.hyper_step(streams, S, H, eps, branch=kinds[0][0], join=join, x_out=streams) is None
    out = torch.empty((2, Hp), dtype=dtype, device="cuda")
    ops.hyper_step(streams, S, H, eps, norm=nw(w), out=out, rows=torch.tensor([3, 0], device="cuda"))
    assert rel(out[:, :H], (ref.rms(xs.sum(0), eps) * w.double())[[3, 0]]) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 20])
@pytest.mark.parametrize("H,Hp", [(90, 96), (520, 520)])
def test_short_convolution_over_portions(dtype, taps, H, Hp):
    """Three sequences in portions of changing sizes, side by side and alone; single tokens go through the fused kernel. Slots are shuffled
    and hold garbage at first; a row without a slot touches none."""
    from inference_b200 import ops

    lens, slots, eps = [70, 33, 5], [3, 0, 5], 1e-3
    u = [rnd(n, H, seed=20 + i) for i, n in enumerate(lens)]           # the normed input, before rounding
    w, nw = rnd(H, taps, seed=4, std=0.6), torch.ones(H)
    h = [ref.rms(t.double(), eps).to(dtype).double() for t in u]
    want = [t + ref.causal_conv(t, w.double()) for t in h]
    pad = lambda t: torch.nn.functional.pad(t, (0, Hp - H)).cuda().contiguous()   # noqa: E731
    conv = ops.ShortConv(pad(w.t()), torch.full((6, taps - 1, Hp), 55.0, dtype=dtype, device="cuda"))
    at = [0, 0, 0]
    got = [[] for _ in lens]
    for cut in ([2, 0, 0], [1, 1, 1], [3, 2, 0], [1, 1, 0], [1, 0, 1], [17, 16, 2], [1, 1, 1], [40, 0, 0], [2, 5, 0], [2, 7, 0]):
        live = [i for i in range(3) if cut[i]]
        one = all(cut[i] == 1 for i in live)
        rows = [(i, p) for i in live for p in range(at[i], at[i] + cut[i])]
        pos, sl = i32([p for _, p in rows]), i32([slots[i] for i in live])
        if one:                      # the fused kernel norms by itself; one stream, read with weight one, and a row without a slot
            x = pad(torch.stack([u[i][p] for i, p in rows] + [u[0][0]]))
            out = torch.empty((len(rows) + 1, Hp), dtype=dtype, device="cuda")
            ops.hyper_step(x, 1, H, eps, norm=ops.NormWeights(pad(nw)), out=out, conv=conv, slots=torch.cat([sl, i32([-1])]),
                           positions=torch.cat([pos, i32([9])]))
            lonely = h[0][0] * (1 + w[:, -1].double())
            assert rel(out[-1, :H], lonely) < OP_TOL[dtype]
            out = out[:-1]
        else:
            x = pad(torch.stack([h[i][p] for i, p in rows]).to(dtype))
            uniform = len({cut[i] for i in live}) == 1
            out = ops.short_conv(x, conv, sl, pos, cu_q=None if uniform else i32([0] + [cut[i] for i in live]).cumsum(0).int(),
                                 max_q_len=max(cut))
        assert (out[:, H:] == 0).all()
        for (i, p), o in zip(rows, out):
            got[i].append(o[:H].cpu())
        at = [a + c for a, c in zip(at, cut)]
    assert at == [70, 33, 5]
    for i in range(3):
        assert rel(torch.stack(got[i]), want[i]) < OP_TOL[dtype]
        assert max(rel(a, b) for a, b in zip(got[i], want[i])) < 2 * OP_TOL[dtype]
        if taps - 1 <= lens[i]:
            assert rel(conv.window[slots[i], :, :H], h[i][lens[i] - taps + 1:]) < OP_TOL[dtype] if taps > 1 else True
    assert (conv.window[[1, 2, 4]] == 55).all()
    # a sequence that starts anew in a used slot, in portions shorter than the window
    a = ops.short_conv(pad(h[2][:2].to(dtype)), conv, i32([3]), i32([0, 1]), cu_q=None, max_q_len=2)
    b = ops.short_conv(pad(h[2][2:4].to(dtype)), conv, i32([3]), i32([2, 3]), cu_q=i32([0, 2]), max_q_len=2)
    assert rel(torch.cat([a, b])[:, :H], want[2][:4]) < OP_TOL[dtype]


# ---- preparation of queries, keys and values ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,rot,E", [(6, 2, 40, 24, 24), (1, 1, 10, 6, 7), (16, 1, 64, 64, 96), (2, 1, 136, 100, 132), (32, 8, 128, 128, 128), (3, 3, 16, 0, 8)])
def test_unit_heads_rotation_and_values_side_by_side(dtype, H, G, D, rot, E):
    from inference_b200 import ops
    from inference_b200.models.nafelix import values_together
    from inference_b200.models.stack import half_pairs

    T, dp, vp, bs, eps, order = 5, up8(D), up8(E), 16, 1e-3, half_pairs(D, rot)
    q, k, v = rnd(T, H, D, seed=1, dtype=dtype) * 2, rnd(T, G, D, seed=2, dtype=dtype) * 0.05, rnd(T, G, E, seed=3, dtype=dtype)
    pos, slots = torch.tensor([0, 1, 40, 7, 63]), torch.tensor([35, 3, 16, -1, 47])
    n = values_together(G, vp)
    lay = lambda t, to: torch.nn.functional.pad(t, (0, to - t.shape[-1]))            # noqa: E731
    nq, nk = H * dp, G * dp
    ang = torch.arange(64, dtype=F)[:, None] * 500.0 ** (-2.0 * torch.arange(rot // 2, dtype=F) / max(rot, 1))
    rope = (ang.cos().float().cuda(), ang.sin().float().cuda()) if rot else None
    for unit in (D, 0):
        buf = torch.cat([lay(q[..., order], dp).reshape(T, nq), lay(k[..., order], dp).reshape(T, nk), lay(v, vp).reshape(T, -1)], 1).cuda()
        kc, vc = torch.zeros((4, G, bs, dp), dtype=dtype, device="cuda"), torch.zeros((4, G // n, bs, n * vp), dtype=dtype, device="cuda")
        ops.row_rope_kv_write(buf, pos.int().cuda(), slots.cuda(), kc, vc, H, G, dp, v_col=nq + nk, rope=rope, unit=unit, eps=eps)
        want = [ref.rotate_halves(t.double(), pos, rot, 500.0) for t in (q, k)]
        if unit:
            want = [ref.rms(t, eps) for t in want]
        back = lambda t, h, d, to: t.reshape(-1, h, to)[..., :d]                      # noqa: E731
        assert rel(back(buf[:, :nq], H, D, dp), want[0][..., order]) < OP_TOL[dtype]
        assert rel(back(buf[:, nq:nq + nk], G, D, dp), want[1][..., order]) < OP_TOL[dtype]
        assert (buf[:, :nq + nk].reshape(T, H + G, dp)[..., D:] == 0).all()
        keys, vals = kc.transpose(1, 2).reshape(-1, G, dp), vc.transpose(1, 2).reshape(-1, G, vp)
        for t in (0, 1, 2, 4):
            assert rel(keys[slots[t], :, :D], want[1][t][..., order]) < OP_TOL[dtype] and torch.equal(vals[slots[t], :, :E].cpu(), v[t])
        assert int((keys != 0).any(-1).any(-1).sum()) == 4 and int((vals != 0).any(-1).any(-1).sum()) == 4


# ---- attention -----------------------------------------------------------------------------------------------------------
def _paged(rows, dtype, heads, bs=16, seed=0):
    """Scatters each sequence's rows [n, G, width] over shuffled pages [page, heads, bs, G width / heads]; unused rows hold large values."""
    need = [(len(r) + bs - 1) // bs for r in rows]
    perm = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    w = rows[0].shape[1] * rows[0].shape[2] // heads
    cache, table = torch.full((len(perm), heads, bs, w), 7.0).to(dtype), torch.zeros((len(rows), max(need) + 2), dtype=torch.int32)
    for s, r in enumerate(rows):
        r = r.reshape(len(r), heads, w)
        for b in range(need[s]):
            table[s, b] = page = perm.pop()
            m = r[b * bs:(b + 1) * bs]
            cache[page, :, :len(m)] = m.transpose(0, 1).to(dtype)
    return cache.cuda(), table.cuda()


def _aligned(q, k, at, scale, score=20.0):
    """The key at position `at` and the last query give a score that takes the whole softmax."""
    u = torch.nn.functional.normalize(rnd(q.shape[-1], seed=99), dim=0)
    if 0 <= at < len(k):
        k[at] = (u * 8).bfloat16().float()
    q[-1] = (u * score / (8 * scale)).bfloat16().float()


def _attention_case(dtype, shape, lens, q_lens, how, window, *, mixed, splits=1, plant=None, uniform=False, scale=None, sink_mean=0.0, with_gate=True):
    """`mixed`: heads exchange their weights, gates per head; else gates per output element. `plant`: distance of the standing-out key from
    the last query."""
    from inference_b200 import ops
    from inference_b200.models.nafelix import values_together

    H, G, D, E = shape
    dp, vp = up8(D), up8(E)
    scale = D ** -0.5 if scale is None else scale
    b16 = lambda *s, seed: rnd(*s, seed=seed, dtype=torch.bfloat16).float()   # noqa: E731
    ks, vs = [b16(n, G, D, seed=10 + i) for i, n in enumerate(lens)], [b16(n, G, E, seed=30 + i) for i, n in enumerate(lens)]
    qs = [b16(n, H, D, seed=50 + i) for i, n in enumerate(q_lens)]
    if plant is not None:
        for q, k in zip(qs, ks):
            _aligned(q, k, len(k) - 1 - plant, scale)
    sink, T = rnd(H, seed=3) + sink_mean, sum(q_lens)
    talk = rnd(H, H, seed=4, std=0.5) + 0.6 * torch.eye(H)
    gate = rnd(T, H if mixed else H * E, seed=5, dtype=torch.bfloat16, std=2.0)
    want = []
    for q, k, v in zip(qs, ks, vs):
        w = ref.attention_weights(q.double(), k.double(), torch.arange(len(k) - len(q), len(k)), scale, window, sink.double())
        want.append(ref.apply_weights(ref.mix_heads(w, talk.double()) if mixed else w, v.double()))
    want = torch.cat(want)
    if with_gate:
        want = want * torch.sigmoid(gate.double()).reshape(T, H, -1)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))     # noqa: E731
    n = values_together(G, vp) if mixed else 1
    kc, table = _paged([pad(k, dp) for k in ks], dtype, G)
    vc, _ = _paged([pad(v, vp) for v in vs], dtype, G // n)
    q, fresh = pad(torch.cat(qs), dp).to(dtype).cuda(), None
    if how == "fresh":
        fresh = pad(torch.cat(ks), dp).to(dtype).cuda(), pad(torch.cat(vs), vp).reshape(T, G // n, n * vp).to(dtype).cuda()
    g = None
    if with_gate:
        g = gate.to(dtype).cuda() if mixed else pad(gate.view(T, H, E), vp).reshape(T, -1).to(dtype).cuda()
        g = torch.nn.functional.pad(g, (0, 16))[:, :g.shape[1]]             # strided rows
    cols = H * G * vp if mixed else H * vp
    if how == "exchange":                                                     # one kernel over all heads, and the merge
        assert ops.exchange_decode_fits(H, G, dp, G // n, n * vp, max(q_lens)) and uniform
        got = ops.exchange_attention(q, kc, vc, table, i32(lens), cu_q=None, max_q_len=max(q_lens), scale=scale, talk=ops.head_mix_weights(talk.cuda(), G),
                                     sink=sink.cuda(), gate=g, window=window, decode=True, num_splits=splits)
        ops.check_status()
        got = got.view(T, H, vp)
        assert (got[..., E:] == 0).all()
        return rel(got[..., :E], want)
    out = torch.full((T, cols + 8), 3.0, dtype=dtype, device="cuda")
    ops.chunk_attention(q, kc, vc, table, i32(lens), cu_q=None if uniform else i32([0] + q_lens).cumsum(0).int(), max_q_len=max(q_lens), scale=scale,
                        window=window, sink=sink.cuda(), decode=how == "decode", num_splits=splits, fresh_kv=fresh, out=out[:, :cols],
                        kernel="simple" if how == "simple" else "auto", all_values=mixed, gate=None if mixed else g)
    ops.check_status()
    assert (out[:, cols:] == 3).all()
    got = out[:, :cols]
    if mixed:
        got = ops.head_mix(got.contiguous().view(T, H, G, vp), ops.head_mix_weights(talk.cuda(), G), gate=g)
    got = got.reshape(T, H, vp)
    assert (got[..., E:] == 0).all()
    return rel(got[..., :E], want)


SHAPES = [(8, 2, 56, 48), (6, 3, 40, 24), (4, 1, 128, 128), (16, 4, 72, 64), (12, 4, 32, 96), (3, 3, 10, 7), (24, 2, 16, 8), (5, 1, 64, 72)]


@pytest.mark.parametrize("mixed", [True, False])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [0, 1, 2, 17, 64, 129])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_window_attention_with_sinks(shape, window, how, mixed):
    lens = [401, 1, 130, 257, 37]
    q_lens = lens if how == "fresh" else [1] * 5 if how == "decode" else [150, 1, 2, 200, 20]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        for splits in (1, 2, 7, 16) if how == "decode" else (1,):
            assert _attention_case(dtype, shape, lens, q_lens, how, window, mixed=mixed, splits=splits, uniform=how == "decode") < 1.5 * OP_TOL[dtype]


@pytest.mark.parametrize("mixed", [True, False])
@pytest.mark.parametrize("window", [1, 15, 16, 17, 40, 63, 64, 65, 128, 200])
@pytest.mark.parametrize("gap", [-1, 0, 1])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_keys_at_the_edge_of_a_window(window, gap, how, mixed):
    """A key that takes the whole softmax of the last query, one inside the edge, at it, or one outside."""
    lens = [385, 130, 64]
    q_lens = lens if how == "fresh" else [40, 1, 17] if how == "context" else [1, 2, 1]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        assert _attention_case(dtype, (4, 2, 48, 40), lens, q_lens, how, window, mixed=mixed, splits=3, plant=window - 1 + gap) < 1.5 * OP_TOL[dtype]


EXCHANGE = SHAPES + [(1, 1, 8, 4), (8, 8, 128, 64), (16, 16, 24, 24), (32, 4, 64, 64), (64, 8, 32, 32), (32, 8, 128, 64), (16, 1, 128, 128)]


@pytest.mark.parametrize("shape", EXCHANGE)
@pytest.mark.parametrize("window", [0, 1, 2, 17, 129])
def test_exchange_decode(shape, window):
    """All heads of a sequence in one CTA: head counts from one to sixty-four, odd groups, several query tokens, any number of splits."""
    lens = [401, 1, 130, 257, 37, 16]
    for splits in (1, 2, 7, 32):
        assert _attention_case(torch.bfloat16, shape, lens, [1] * 6, "exchange", window, mixed=True, splits=splits, uniform=True) < 1.5 * OP_TOL[torch.bfloat16]
    if shape[0] * 3 <= 16:
        for splits in (1, 5):
            assert _attention_case(torch.bfloat16, shape, [401, 3, 130], [3] * 3, "exchange", window, mixed=True, splits=splits, uniform=True) < 1.5 * OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("window", [1, 15, 16, 17, 40, 64, 128, 200])
@pytest.mark.parametrize("gap", [-1, 0, 1])
def test_exchange_decode_at_the_edge_of_a_window(window, gap):
    for q in (1, 2):
        assert _attention_case(torch.bfloat16, (4, 2, 48, 40), [385, 130, 64], [q] * 3, "exchange", window, mixed=True, splits=3, plant=window - 1 + gap,
                               uniform=True) < 1.5 * OP_TOL[torch.bfloat16]
    for mean in (8.0, -30.0):
        assert _attention_case(torch.bfloat16, (8, 4, 32, 64), [300, 70], [2, 2], "exchange", window, mixed=True, splits=4, uniform=True,
                               sink_mean=mean, with_gate=gap > 0) < 2 * OP_TOL[torch.bfloat16]


def test_exchange_decode_limits_agree():
    from inference_b200 import ops
    from inference_b200._native import kernels

    g = torch.Generator().manual_seed(0)
    yes = 0
    for _ in range(3000):
        G, D, NV, Dv, q = (int(torch.randint(1, n, (1,), generator=g)) for n in (18, 18, 18, 18, 4))
        H = G * int(torch.randint(1, 9, (1,), generator=g))
        fits = ops.exchange_decode_fits(H, G, D * 8, NV, Dv * 8, q)
        assert fits == (kernels().swb_exchange_decode_stages(H, G, D * 8, NV, Dv * 8, q) > 0)
        yes += fits
    assert 100 < yes < 2900


@pytest.mark.parametrize("mixed", [True, False])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_sinks_far_above_and_below_the_scores(how, mixed):
    """Far keys without a window, portions of a few tokens each, sinks that take everything or nothing, no gate, a scale below zero."""
    lens = [300, 70]
    q_lens = lens if how == "fresh" else [2, 2] if how == "decode" else [40, 3]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        for mean in (8.0, -30.0):
            assert _attention_case(dtype, (8, 4, 32, 64), lens, q_lens, how, 0, mixed=mixed, splits=2, uniform=how == "decode", sink_mean=mean) < 2 * OP_TOL[dtype]
        assert _attention_case(dtype, (8, 4, 32, 64), lens, q_lens, how, 90, mixed=mixed, plant=250, with_gate=False, sink_mean=2.0) < 2 * OP_TOL[dtype]
    assert _attention_case(torch.bfloat16, (2, 1, 16, 16), [70, 66], [2, 2], how if how != "fresh" else "context", 9, mixed=mixed, scale=-0.2) < 2 * OP_TOL[torch.bfloat16]
    assert _attention_case(torch.bfloat16, (4, 2, 136, 144), [70, 66], [3, 2], "context", 30, mixed=mixed) < 2 * OP_TOL[torch.bfloat16]   # plain kernel


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,G,Dv", [(1, 1, 1, 8), (5, 6, 3, 24), (600, 10, 2, 40), (7, 40, 2, 64), (513, 24, 24, 8), (3, 32, 4, 128)])
def test_heads_exchange_weights(dtype, T, H, G, Dv):
    from inference_b200 import ops

    a, talk, gate = rnd(T, H, G, Dv, seed=1, dtype=dtype), rnd(H, H, seed=2), rnd(T, H + 3, seed=3, dtype=dtype)[:, :H]
    want = torch.stack([sum(talk[h, g].double() * a[:, g, h // (H // G)].double() for g in range(H)) for h in range(H)], 1)
    tw = ops.head_mix_weights(talk.cuda(), G)
    assert rel(ops.head_mix(a.cuda(), tw), want.reshape(T, -1)) < OP_TOL[dtype]
    assert rel(ops.head_mix(a.cuda(), tw, gate=gate.cuda()), (want * torch.sigmoid(gate.double())[..., None]).reshape(T, -1)) < OP_TOL[dtype]


# ---- delta rule ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,E,taps", [(4, 2, 32, 64, 4), (6, 2, 24, 40, 3), (1, 1, 5, 9, 2), (3, 3, 100, 24, 1), (4, 2, 128, 128, 4), (2, 1, 200, 16, 6),
                                          (2, 2, 300, 8, 4), (8, 4, 64, 136, 4)])
def test_delta_rule_with_one_decay_per_head(dtype, H, G, D, E, taps):
    """Convolutions, decays, the recurrence, norm and gate over portions of two sequences (single tokens too), against the whole sequence;
    states and windows in shuffled slots that hold garbage at first."""
    from inference_b200 import ops

    dp, vp, hb, eps = ops.delta_key_width(D), up8(E), up8(H), 1e-3
    lens, slots = [75, 31], [2, 0]
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))     # noqa: E731
    conv = [rnd(n, taps, seed=s, std=0.6) for n, s in ((G * D, 1), (G * D, 2), (H * E, 3))]
    a_log, dt, nw = rnd(H, seed=4) * 0.5 - 1, rnd(H, seed=5) * 0.5 - 1.5, rnd(E, seed=6) * 0.3 + 1
    want, rows = [], []
    for i, n in enumerate(lens):
        q, k, v, z = (rnd(n, c, seed=10 * i + s, dtype=dtype) for c, s in ((G * D, 11), (G * D, 12), (H * E, 13), (H * E, 14)))
        b, a = rnd(n, H, seed=10 * i + 15, dtype=dtype), rnd(n, H, seed=10 * i + 16, dtype=dtype)
        c = [ref.silu(ref.causal_conv(t.double(), w.double())) for t, w in zip((q, k, v), conv)]
        o, state = ref.delta_rule(ref.unit(c[0].view(n, G, D)) * D ** -0.5, ref.unit(c[1].view(n, G, D)), c[2].view(n, H, E),
                                  ref.head_decay(a.double(), a_log.double(), dt.double()), torch.sigmoid(b.double()))
        want.append((ref.rms(o, eps) * nw.double() * ref.silu(z.double()).view(n, H, E), state))
        rows.append(torch.cat([pad(q.view(n, G, D), dp).reshape(n, -1), pad(k.view(n, G, D), dp).reshape(n, -1), pad(v.view(n, H, E), vp).reshape(n, -1),
                               pad(b, hb), pad(a, hb), pad(z.view(n, H, E), vp).reshape(n, -1)], 1))
    cw = torch.cat([pad(w.view(h, d, taps).transpose(1, 2), to).permute(1, 0, 2).reshape(taps, -1)
                    for w, h, d, to in zip(conv, (G, G, H), (D, D, E), (dp, dp, vp))], 1)
    col_b = 2 * G * dp + H * vp
    w = ops.DeltaWeights(H, G, D, dp, E, vp, col_b, cw.cuda().contiguous(), a_log.cuda(), dt.cuda(), pad(nw, vp).cuda(), head_decay=True, col_a=col_b + hb)
    state = torch.full((3, *w.state_shape()), 9.0, device="cuda")
    window = torch.full((3, *w.window_shape()), 9.0, dtype=dtype, device="cuda")
    at, got = [0, 0], [[], []]
    for cut in ([2, 0], [1, 1], [3, 2], [1, 1], [16, 1], [33, 17], [1, 1], [18, 8]):
        live = [i for i in (0, 1) if cut[i]]
        buf = torch.cat([rows[i][at[i]:at[i] + cut[i]] for i in live]).cuda()
        pos = i32([p for i in live for p in range(at[i], at[i] + cut[i])])
        uniform = len({cut[i] for i in live}) == 1
        out = ops.head_delta(buf, buf[:, col_b + 2 * hb:], w, eps, state, window, i32([slots[i] for i in live]), pos,
                             cu_q=None if uniform else i32([0] + [cut[i] for i in live]).cumsum(0).int(), max_q_len=max(cut))
        o = 0
        for i in live:
            got[i].append(out[o:o + cut[i]].view(-1, H, vp).cpu())
            o, at[i] = o + cut[i], at[i] + cut[i]
    assert at == lens
    for i in (0, 1):
        g = torch.cat(got[i])
        assert rel(g[..., :E], want[i][0]) < 2 * OP_TOL[dtype] and (g[..., E:] == 0).all()
        assert rel(state[slots[i], :, :E, :D].transpose(1, 2), want[i][1]) < 2 * OP_TOL[dtype]
    assert (state[1] == 9).all() and (window[1] == 9).all()


# ---- feed-forward --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,N,K", [(1, 24, 64), (5, 136, 1024), (64, 520, 2048), (100, 128, 256), (300, 384, 256), (1000, 1024, 512)])
def test_xielu_in_the_epilogue(T, N, K):
    from inference_b200 import ops

    a, w, pq = rnd(T, K, seed=1, dtype=torch.bfloat16), rnd(N, K, seed=2, dtype=torch.bfloat16, std=2 * K ** -0.5), torch.tensor([0.4, -0.9])
    a[0] *= 0.01                                         # around zero, where the two branches meet
    want = ref.xielu(a.double() @ w.double().T, pq.double())
    prm = (float(ref.softplus(pq[0])), 0.5 + float(ref.softplus(pq[1])))
    assert rel(ops.gemm_bf16(a.cuda(), w.cuda(), act="xielu", act_params=prm), want) < 4e-3
    wide = ops.gemm_bf16(a.cuda(), w.cuda(), act="xielu", act_params=prm, out_dtype=torch.float32)
    assert rel(wide, want) < 2e-5 and rel(wide[0], want[0]) < 1e-4
    assert rel(ops.gemm_f32(a.float().cuda(), w.float().cuda(), act="xielu", act_params=prm), want) < 2e-6
    z = torch.linspace(-30, 30, 4001)
    eye = torch.zeros(8)
    eye[0] = 1.0
    got = ops.gemm_f32((z[:, None] * eye).cuda(), torch.eye(8).cuda(), act="xielu", act_params=prm)[:, 0]
    assert rel(got, ref.xielu(z.double(), pq.double())) < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("limit", [0.3, 1.0, 7.0])
def test_clamped_gated_units(dtype, limit):
    from inference_b200 import ops

    T, ff = 7, 72
    g, u = rnd(T, ff, seed=1, dtype=dtype) * 3, rnd(T, ff, seed=2, dtype=dtype) * 3
    eye = torch.eye(ff, dtype=F)
    want = torch.stack([torch.clamp(g.double(), max=limit), torch.clamp(u.double(), -limit, limit)])
    want = want[0] * torch.sigmoid(1.702 * want[0]) * (want[1] + 1)
    assert float((ref.clamped_expert(g.double(), eye, torch.zeros(ff, ff, dtype=F), eye, limit) - torch.clamp(g.double(), max=limit) * torch.sigmoid(
        1.702 * torch.clamp(g.double(), max=limit))).abs().max()) < 1e-12
    assert rel(ops.gated_act_mul(torch.stack([g, u], -1).reshape(T, -1).cuda(), "clamped", paired=True, limit=limit), want) < OP_TOL[dtype]
    assert rel(ops.gated_act_mul(torch.cat([g, u], 1).cuda(), "clamped", limit=limit), want) < OP_TOL[dtype]
    if dtype == torch.bfloat16:                          # in the epilogue of a decode-sized projection
        x, w = rnd(5, 512, seed=3, dtype=dtype), rnd(64, 512, seed=4, dtype=dtype, std=3 * 512 ** -0.5)
        z = x.double() @ w.double().T
        got = ops.gemm_bf16(x.cuda(), w.cuda(), act="clamped_pairs", act_params=(limit, 0.0))
        zg, zu = torch.clamp(z[:, ::2], max=limit), torch.clamp(z[:, 1::2], -limit, limit)
        assert rel(got, zg * torch.sigmoid(1.702 * zg) * (zu + 1)) < OP_TOL[dtype]


@pytest.mark.parametrize("dtype,padded", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
@pytest.mark.parametrize("T,E,top,W,ff", [(1, 4, 2, 96, 24), (40, 6, 3, 64, 56), (70, 3, 3, 256, 136), (200, 40, 1, 64, 24), (9, 64, 40, 64, 16)])
def test_routed_clamped_experts(dtype, padded, T, E, top, W, ff):
    """Chosen scores divided by their sum; clamped units; every kernel that serves a step size."""
    from inference_b200 import ops

    h, g, u, d = rnd(T, W, seed=1, dtype=dtype), *(rnd(E, ff, W, seed=s, std=2 * W ** -0.5, dtype=dtype) for s in (2, 3)), rnd(E, W, ff, seed=4, std=ff ** -0.5, dtype=dtype)
    router = rnd(E, W, seed=5, std=2 * W ** -0.5)
    e, w = ref.route(h.double(), router.double(), top)
    assert torch.allclose(w.sum(-1), torch.ones(T, dtype=F))
    want = torch.zeros(T, W, dtype=F)
    for t in range(T):
        for j in range(top):
            x = int(e[t, j])
            want[t] += w[t, j] * ref.clamped_expert(h[t].double(), g[x].double(), u[x].double(), d[x].double(), 0.9)
    z = (h.double() @ router.double().T).float()
    for _ in range(2):                                   # twice: the routing counters clear themselves
        plan, rows = ops.logits_routing(z.cuda(), E, top, rows=h.cuda() if padded else None, renorm=True)
        assert rel(plan.weights, w) < 1e-5
        pairs = torch.stack([g, u], 2).reshape(E, 2 * ff, W).cuda()
        y = ops.routed_gated_ffn(rows if padded else h.cuda(), pairs, d.cuda(), plan, "clamped", 0.9)
        got = (y.float()[plan.dest.long()] * plan.weights[..., None]).sum(1)
        assert rel(got, want) < OP_TOL[dtype]


# ---- whole models --------------------------------------------------------------------------------------------------------
_CACHE: dict = {}


def _model(name):
    if name not in _CACHE:
        cfg = ref.MODELS[name]()
        _CACHE[name] = (cfg, ref.random_weights(cfg, seed=ord(name)), {})
    return _CACHE[name]


def _tokens(name, n, seed=0):
    return torch.randint(0, _model(name)[0]["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _want(name, tokens):
    """(logits, sums of the streams after every layer run, smallest router margin [T])"""
    cfg, w, memo = _model(name)
    key = tuple(tokens)
    if key not in memo:
        taps, margins = [], []
        logits = ref.forward(cfg, w, tokens, taps, margins)
        memo[key] = logits, taps, torch.stack(margins).min(0).values
    return memo[key]


def _sure(name, tokens, gap=0.15):
    """Rows whose experts are no close call: rounding h to bf16 cannot choose others."""
    return _want(name, tokens)[2] > gap


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
    return backend.runner.pool.allocator.live_blocks() == 0 and backend.runner.pool.slots.live_blocks() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ref.MODELS))
def test_every_layer_run_matches(name, dtype):
    b = _backend(name, dtype)
    model, tokens, got = b.runner.model, _tokens(name, 60, 1), []
    fwd = model.forward_hidden
    model.forward_hidden = lambda inp, kv: fwd(inp, kv, tap=got.append)
    b.forward_at([b.new_sequence()], [tokens], [[0]])
    _, trail, margins = _want(name, tokens)
    assert len(got) == len(trail) == len(ref.runs(_model(name)[0]))
    sure = margins > (0.15 if dtype == torch.bfloat16 else 0.0)
    for i, (x, y) in enumerate(zip(got, trail)):
        assert rel(x.cpu()[sure], y[sure]) < (TOL[dtype] if dtype == torch.float32 else 2 * TOL[dtype]), (i, rel(x.cpu()[sure], y[sure]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ref.MODELS))
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [3, 2, 7, 16, 17, 31], [64], [100, 1]])
def test_prompts_portions_and_decoding_agree(name, dtype, cuts):
    """Whole prompt, token by token (graph-replayed decode), and portions from two tokens up give the same logits."""
    tokens = _tokens(name, 139, 2)
    b = _backend(name, dtype)
    got = _feed(b, b.new_sequence(), tokens, list(cuts))
    want, sure = _want(name, tokens)[0], _sure(name, tokens)
    if dtype == torch.float32:
        assert rel(got, want) < TOL[dtype] and max(rel(g, w) for g, w in zip(got, want)) < 4 * TOL[dtype]
        return
    assert int(sure.sum()) > 30
    assert rel(got.cpu()[sure], want[sure]) < 2 * TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_agree_with_the_whole_prompt_closely(dtype):
    """The same kernels' rounding apart, a position's logits do not depend on the cuts: tighter than against the restatement."""
    tokens = _tokens("d", 200, 8)
    b = _backend("d", dtype)
    whole = _feed(b, b.new_sequence(), tokens, [1000])
    sure = _sure("d", tokens)
    for cuts in ([37, 2, 3, 64, 1, 1, 50, 2], [150, 1], [1, 1, 1, 120, 1]):
        got = _feed(b, b.new_sequence(), tokens, list(cuts))
        assert rel(got.cpu()[sure], whole.cpu()[sure]) < (1e-5 if dtype == torch.float32 else TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_contexts_decode_with_split_kv(dtype):
    tokens = _tokens("d", 700, 3)
    want, sure = _want("d", tokens)[0], _sure("d", tokens)
    b = _backend("d", dtype, ctx=800, kv_tokens=704)
    got = _feed(b, b.new_sequence(), tokens, [480, 50, 5, 12, 1])
    keep = sure if dtype == torch.bfloat16 else torch.ones_like(sure)
    tol = TOL[dtype] * (2 if dtype == torch.bfloat16 else 1)
    assert rel(got.cpu()[keep], want[keep]) < tol and rel(got.cpu()[-150:][keep[-150:]], want[-150:][keep[-150:]]) < tol
    assert max(b.runner.model.decode_splits(1, 700)) > 1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "c"])
def test_mixed_batches_and_reused_pages_and_slots(name, dtype):
    """Portions of some sequences beside single tokens of others, sequences that pause, end and give their pages and slots to new ones;
    both are just enough. Every logit equals that of the sequence alone."""
    lens = {"p": 90, "q": 33, "r": 150, "s": 17, "t": 120, "u": 64}
    toks = {k: _tokens(name, n, 10 + i) for i, (k, n) in enumerate(lens.items())}
    b = _backend(name, dtype, max_batch=4, ctx=160, kv_tokens=352)
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
        keep = _sure(name, toks[k]) if dtype == torch.bfloat16 else torch.ones(lens[k], dtype=torch.bool)
        assert rel(torch.cat(got[k]).cpu()[keep], _want(name, toks[k])[0][keep]) < TOL[dtype] * (2 if dtype == torch.bfloat16 else 1), k


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

    slack = 1e-4 if dtype == torch.float32 else 0.5
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
    assert generate(_backend("b", torch.float32), prompt, GenerationConfig(max_new_tokens=10)).tokens == ref.greedy(cfg, w, prompt, 10)


@pytest.mark.parametrize("dtype", DTYPES)
def test_large_batches_pad_to_a_bucket(dtype):
    """19 rows decode in a graph captured for 24; the padding rows change nothing, nor does the capture's warm-up move a state."""
    b = _backend("b", dtype, max_batch=24, ctx=64, kv_tokens=24 * 64)
    toks = [_tokens("b", 12 + i, 100 + i) for i in range(19)]
    seqs = [b.new_sequence() for _ in toks]
    b.forward_at(seqs, [t[:-3] for t in toks], [[] for _ in toks])
    for back in (3, 2, 1):
        got = b.forward_at(seqs, [[t[-back]] for t in toks], [[0] for _ in toks])
        for g, t in zip(got, toks):
            if dtype == torch.float32 or _sure("b", t)[-back]:
                assert rel(g, _want("b", t)[0][-back]) < (TOL[dtype] if dtype == torch.float32 else 4 * TOL[dtype])


# ---- provider and replay tool ---------------------------------------------------------------------------------------------
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
    assert llm.descriptor().family == "nafelix"
    req = TextLlmRequest(messages=[Message.user("hello world the cat")], max_new_tokens=8, sampling=Sampling(temperature=0.0))
    events = []
    out = llm.generate(req, events.append)
    assert 0 < out.usage.generated_tokens <= 8 and events
    hot = TextLlmRequest(messages=[Message.user("hello world the cat")], max_new_tokens=8, seed=3,
                         sampling=Sampling(temperature=0.9, top_p=0.9))
    assert llm.generate(hot, lambda e: None).text == llm.generate(hot, lambda e: None).text


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_replays_steps(tmp_path, dtype):
    d, out = _snapshot(tmp_path / "m", "d"), tmp_path / "out"
    x, y = _tokens("d", 80, 6), _tokens("d", 45, 7)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": x[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": x[50:51], "want": [0]}, {"id": "y", "tokens": y, "want": [44]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": x[51:52], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "x", "tokens": x[52:], "want": [27, 1]}], "end": ["x"]}]
    r = subprocess.run([sys.executable, str(Path(__file__).resolve().parent.parent / "bin" / "trace_run"), "--model", str(d),
                        "--dtype", dtype, "--out", str(out), "--max-tokens", "144"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    wx, wy = _want("d", x)[0], _want("d", y)[0]
    want = {0: wx[[0, 49]], 1: torch.stack([wx[50], wy[44]]), 3: wx[[79, 53]]}
    assert sorted(p.name for p in out.iterdir()) == [f"{i}.f32" for i in want]
    for i, w in want.items():
        got = torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(len(w), -1)
        if dtype == "float32":
            assert rel(got, w) < TOL[torch.float32]
        else:
            assert rel(got, w) < 0.2
