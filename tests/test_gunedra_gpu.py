"""Gunedra on the GPU against the plain float64 restatement in tests/gunedra_reference.py: each mechanism alone, then whole
models in float32 and bfloat16 through the runner, the paged pool with its state slots, the generation loops, the provider and
the replay tool."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import gunedra_reference as ref

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


# ---- stream: grouped norms, depth average, scaled embedding -----------------------------------------------------------
@pytest.mark.parametrize("H,Hp,groups", [(160, 160, 5), (90, 96, 3), (9, 16, 9), (256, 256, 2), (384, 384, 3), (2048, 2048, 2), (4096, 4096, 32),
                                         (9000, 9000, 4), (512, 512, 1), (30, 32, 1)])
def test_group_norm_joins_and_depth_average(H, Hp, groups):
    from inference_b200 import ops

    T, eps, n = 5, 1e-2, 3
    pad = lambda t: torch.nn.functional.pad(t, (0, Hp - H)).cuda().contiguous()   # noqa: E731
    x, y, w1, w2 = rnd(T, H, seed=1), rnd(T, H, seed=2) * torch.linspace(0.1, 4, H), rnd(H, seed=3), rnd(H, seed=4)
    earlier, mix = rnd(n, T, H, seed=5), rnd(n + 1, seed=6)
    d = [t.double() for t in (x, y, w1, w2, earlier, mix)]
    joined = d[0] + ref.grouped_norm(d[1], d[2], groups, eps)
    kw = dict(center=False, groups=groups)
    gx, out = pad(x), torch.full((T, Hp), 9.0, device="cuda")
    ops.stream_norm(gx, H, eps, branch=ops.Branch(pad(y), ops.NormWeights(pad(w1))), norm=ops.NormWeights(pad(w2)), out=out, **kw)
    assert rel(gx[:, :H], joined) < 1e-6 and rel(out[:, :H], ref.grouped_norm(joined, d[3], groups, eps)) < 2e-6
    # read from elsewhere, file as result n, go on with the average; bf16 copy of it
    res = torch.zeros((n + 1, T, Hp), device="cuda")
    res[:n, :, :H] = earlier.cuda()
    gx, copy = torch.full((T, Hp), 5.0, device="cuda"), torch.empty((T, Hp), device="cuda", dtype=torch.bfloat16)
    ops.stream_norm(gx, H, eps, branch=ops.Branch(pad(y), ops.NormWeights(pad(w1))), out=copy, x_in=pad(x),
                    average=ops.DepthAverage(res, n, mix.cuda()), **kw)
    avg = ref.depth_average([*d[4], joined], d[5])
    assert rel(res[n, :, :H], joined) < 1e-6 and rel(gx[:, :H], avg) < 2e-6 and rel(copy[:, :H], avg) < 4e-3
    assert torch.equal(res[:n, :, :H].cpu(), earlier)
    # chosen rows, no branch
    out = torch.empty((2, Hp), device="cuda")
    ops.stream_norm(pad(x), H, eps, norm=ops.NormWeights(pad(w2)), out=out, rows=torch.tensor([3, 0], device="cuda"), **kw)
    assert rel(out[:, :H], ref.grouped_norm(d[0], d[3], groups, eps)[[3, 0]]) < 2e-6


def test_scaled_embedding():
    from inference_b200 import ops

    table, ids = rnd(30, 24, dtype=torch.bfloat16).cuda(), torch.tensor([4, 29, 0, 4], device="cuda")
    h = torch.empty((4, 24), dtype=torch.bfloat16, device="cuda")
    x = ops.stream_embed(ids, table, copies=[h], scale=1.7)
    assert torch.equal(x, table.float()[ids] * 1.7) and torch.equal(h, x.bfloat16())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,fp", [(1, 8), (13, 16), (384, 384), (2050, 2056), (8448, 8448), (12000, 12000), (17000, 17000)])
def test_poly_norm(dtype, ff, fp):
    from inference_b200 import ops

    z, coef = rnd(3, ff, dtype=dtype) * torch.tensor([[0.01], [1.0], [30.0]]).to(dtype), torch.tensor([0.7, -0.4, 0.3, 0.2])
    got = ops.poly_norm(torch.nn.functional.pad(z, (0, fp - ff)).cuda(), coef.cuda(), 1e-3, ff)
    for r in range(3):
        assert rel(got[r, :ff], ref.poly_norm(z[r].double(), coef.double(), 1e-3)) < (2e-6 if dtype == torch.float32 else 4e-3)


# ---- latent attention ---------------------------------------------------------------------------------------------------
def _weights(H, dim, rot, vdim, rank, dtype=torch.bfloat16, scale=None, seed=0, sink_mean=0.0):
    """(LatentWeights with padding, plain uk, plain uv)."""
    from inference_b200 import ops

    up = lambda n, m: (n + m - 1) // m * m   # noqa: E731
    dn, rp, rk, vp = up(dim, 16), up(rot, 8), up(rank, 64), up(vdim, 16)
    uk, uv = (rnd(H, d, rank, seed=seed + s, dtype=torch.bfloat16, std=rank ** -0.5) for s, d in ((1, dim), (2, vdim)))
    pad = lambda t, n: torch.nn.functional.pad(t, (0, rk - rank, 0, n - t.shape[1])).to(dtype).cuda()   # noqa: E731
    ku, vu = pad(uk, dn), pad(uv, vp)
    w = ops.LatentWeights(H, dim, dn, rot, rp, rank, rk, vdim, vp, (dim + rot) ** -0.5 if scale is None else scale,
                          torch.nn.functional.pad(rnd(rank, seed=seed + 3), (0, rk - rank)).cuda(), (rnd(H, seed=seed + 4) + sink_mean).cuda(),
                          torch.cat([ku.reshape(H * dn, rk), vu.reshape(H * vp, rk)]), ku.transpose(1, 2).contiguous())
    return w, uk.double(), uv.double()


def _rows(w, c, kr):
    """Cached rows [c | k_rot] with padding."""
    out = torch.zeros(c.shape[0], w.width)
    out[:, :w.rank], out[:, w.rk:w.rk + w.rot] = c, kr
    return out


def _paged(rows, dtype, bs=16, seed=0):
    """Scatters each sequence's rows over shuffled pages; unused page rows hold large values."""
    need = [(len(r) + bs - 1) // bs for r in rows]
    perm = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    cache, table = torch.full((len(perm), bs, rows[0].shape[1]), 7.0).to(dtype), torch.zeros((len(rows), max(need) + 2), dtype=torch.int32)
    for s, r in enumerate(rows):
        for b in range(need[s]):
            table[s, b] = page = perm.pop()
            m = r[b * bs:(b + 1) * bs]
            cache[page, :len(m)] = m.to(dtype)
    return cache.cuda(), table.cuda()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,rot,rank", [(3, 40, 24, 96), (1, 18, 6, 20), (16, 128, 64, 512), (2, 16, 72, 600)])
def test_latent_prep_norms_rotates_and_writes(dtype, H, dim, rot, rank):
    from inference_b200 import ops

    w, _, _ = _weights(H, dim, rot, 16, rank, dtype)
    T, bs, eps = 5, 16, 1e-3
    pos, slots = torch.tensor([0, 1, 40, 7, 63]), torch.tensor([35, 3, 16, -1, 47])
    q, low = rnd(T, H, dim + rot, seed=1, dtype=dtype), rnd(T, rank + rot, seed=2, dtype=dtype) * 3
    proj = torch.zeros(T, w.col_gate + 8, dtype=dtype)
    pq = proj[:, :w.col_c].view(T, H, w.dn + w.rp)
    pq[..., :dim], pq[..., w.dn:w.dn + rot] = q[..., :dim], q[..., dim:]
    proj[:, w.col_c:w.col_c + rank], proj[:, w.col_c + w.rk:w.col_c + w.rk + rot] = low[:, :rank], low[:, rank:]
    ang = torch.arange(64, dtype=F)[:, None] * 300.0 ** (-2.0 * torch.arange(rot // 2, dtype=F) / rot)
    cache, buf = torch.zeros((4, bs, w.width), dtype=dtype, device="cuda"), proj.cuda()
    q_abs = torch.zeros((3, H, w.width), dtype=dtype, device="cuda")
    ops.latent_prep(buf, w, eps, ang.cos().float().cuda(), ang.sin().float().cuda(), pos.int().cuda(), slots.cuda(), cache, q_abs,
                    i32([2, -1, 0, 1, -1]))
    c = ref.rms(low[:, :rank].double(), eps) * w.norm[:rank].double().cpu()
    kr = ref.rotate_pairs(low[:, None, rank:].double(), pos, rot, 300.0)[:, 0]
    qr = ref.rotate_pairs(q[..., dim:].double(), pos, rot, 300.0)
    out = buf[:, :w.col_c].view(T, H, w.dn + w.rp)
    assert torch.equal(out[..., :dim].cpu(), q[..., :dim]) and rel(out[..., w.dn:w.dn + rot], qr) < OP_TOL[dtype]
    assert rel(buf[:, w.col_c:w.col_c + rank], c) < OP_TOL[dtype]
    flat = cache.view(-1, w.width)
    for t in (0, 1, 2, 4):
        assert rel(flat[slots[t], :rank], c[t]) < OP_TOL[dtype] and rel(flat[slots[t], w.rk:w.rk + rot], kr[t]) < OP_TOL[dtype]
    assert int((flat != 0).any(-1).sum()) == 4                  # the token without a slot wrote nothing
    for row, t in enumerate((2, 3, 0)):
        assert rel(q_abs[row, :, w.rk:w.rk + rot], qr[t]) < OP_TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,N,K", [(1, 4, 64, 16), (5, 3, 24, 40), (33, 16, 512, 128), (17, 2, 128, 640)])
def test_head_products(dtype, T, H, N, K):
    from inference_b200 import ops

    a, w, gate = rnd(T, H, K + 8, seed=1, dtype=dtype), rnd(H, N, K, seed=2, dtype=dtype, std=K ** -0.5), rnd(T, H + 3, seed=3, dtype=dtype)
    want = torch.einsum("thk,hnk->thn", a[..., :K].double(), w.double())
    out = torch.empty((T, H, N + 8), dtype=dtype, device="cuda")[..., :N]
    ops.head_product(a.cuda()[..., :K], w.cuda(), out)
    assert rel(out, want) < OP_TOL[dtype]
    ops.head_product(a.cuda()[..., :K], w.cuda(), out, gate=gate.cuda()[:, :H])
    gated = want * torch.sigmoid(gate[:, :H].double())[..., None]
    assert rel(out, gated) < OP_TOL[dtype]
    if dtype == torch.bfloat16 and T > 4:
        ops.head_product(a.cuda()[..., :K], w.cuda(), out, kernel="simple")
        assert rel(out, want) < OP_TOL[dtype]
        out.zero_()
        ops.head_product(a.cuda()[..., :K], w.cuda(), out, gate=gate.cuda()[:, :H], rows_in=i32([4, 0]), rows_out=i32([1, 3]))
        both = want[[4, 0]] * torch.sigmoid(gate[[1, 3], :H].double())[..., None]
        assert rel(out[[1, 3]], both) < OP_TOL[dtype] and int((out != 0).any(-1).any(-1).sum()) == 2


def _latent_case(dtype, H, dim, rot, vdim, rank, lens, q_lens, how, splits=1, bs=16, scale=None, sink_mean=0.0, plant=None, listed=None,
                 uniform=False):
    """Attention of the last q_lens[i] tokens of every sequence through latent rows, gate included. `plant`: the last query of
    every sequence is aligned with the key at that position, which then takes nearly all of its weight."""
    from inference_b200 import ops

    w, uk, uv = _weights(H, dim, rot, vdim, rank, dtype, scale, sink_mean=sink_mean)
    cs = [rnd(n, rank, seed=10 + i, dtype=torch.bfloat16).float() for i, n in enumerate(lens)]
    krs = [rnd(n, rot, seed=30 + i, dtype=torch.bfloat16).float() for i, n in enumerate(lens)]
    qs = [rnd(n, H, dim + rot, seed=50 + i, dtype=torch.bfloat16).float() for i, n in enumerate(q_lens)]
    if plant is not None:
        for kr, q, n in zip(krs, qs, lens):
            at = plant if plant >= 0 else n + plant
            if 0 <= at < n:
                u = torch.nn.functional.normalize(rnd(rot, seed=99), dim=0)
                kr[at], q[-1, :, dim:] = (u * 8).bfloat16().float(), (u * 20.0 / (8 * w.scale)).bfloat16().float()
    T = sum(q_lens)
    gate = rnd(T, H, seed=8, dtype=torch.bfloat16)
    want = []
    for c, kr, q, n in zip(cs, krs, qs, lens):
        k, v = ref.latent_keys_values(c.double(), kr.double(), uk.reshape(-1, rank), uv.reshape(-1, rank), H)
        want.append(ref.sink_attention(q.double(), k, v, torch.arange(n - len(q), n), w.scale, w.sink.double().cpu()))
    want = torch.cat(want) * torch.sigmoid(gate.double())[..., None]
    rows = [_rows(w, c, kr) for c, kr in zip(cs, krs)]
    cache, table = _paged(rows, dtype, bs)
    q = torch.zeros(T, H, w.dn + w.rp)
    q[..., :dim], q[..., w.dn:w.dn + rot] = torch.cat(qs)[..., :dim], torch.cat(qs)[..., dim:]
    q, g, out = q.to(dtype).cuda(), gate.to(dtype).cuda(), torch.zeros((T, H, w.vp), dtype=dtype, device="cuda")
    cu = i32([0] + q_lens).cumsum(0).int()
    keep = slice(None)
    if how in ("decode", "simple"):
        q_abs = torch.empty((T, H, w.width), dtype=dtype, device="cuda")
        q_abs[..., w.rk:] = torch.nn.functional.pad(q[..., w.dn:], (0, w.rc - w.rp))
        ops.head_product(q[..., :w.dn], w.uk_t, q_abs[..., :w.rk])
        kw = dict(cu_q=None if uniform else cu, max_q_len=max(q_lens))
        lat = ops.latent_decode(q_abs, cache, table, i32(lens), w, num_splits=splits, **kw) if how == "decode" else \
            ops.latent_attention_simple(q_abs, cache, table, i32(lens), w, **kw)
        ops.head_product(lat, w.uv, out, gate=g, sink=w.sink)
    else:
        kw, ids = {}, listed or list(range(len(lens)))
        flat = torch.cat(rows).to(dtype).cuda()
        if how == "context":
            flat = ops.latent_gather(cache, table, i32([0] + [lens[i] for i in ids]).cumsum(0).int(), sum(lens[i] for i in ids), i32(ids))
            assert torch.equal(flat.cpu(), torch.cat([rows[i] for i in ids]).to(dtype))
            kw = dict(seqs=i32(ids), cu_k=i32([0] + [lens[i] for i in ids]).cumsum(0).int())
            starts = [0] + torch.tensor(q_lens).cumsum(0).tolist()
            keep = [t for i in ids for t in range(starts[i], starts[i + 1])]
        kv = ops.gemm_bf16(flat[:, :w.rk], w.ukv)
        ops.latent_prefill(q.view(T, -1), kv, flat[:, w.rk:w.rk + w.rp], w, out.view(T, -1), cu_q=cu, max_q_len=max(q_lens[i] for i in ids), gate=g, **kw)
        rest = [t for t in range(T) if how == "context" and t not in keep]
        assert (out[rest] == 0).all()
    ops.check_status()
    return rel(out[keep][..., :vdim], want[keep])


SHAPES = [(4, 64, 16, 64, 128), (3, 40, 24, 56, 96), (16, 128, 64, 128, 512), (20, 32, 32, 48, 192), (1, 18, 6, 14, 20), (40, 16, 8, 24, 64),
          (5, 24, 96, 16, 320)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("splits", [1, 2, 7, 32])
def test_latent_decode(shape, splits):
    lens = [1, 16, 17, 64, 65, 300, 1023]
    assert _latent_case(torch.bfloat16, *shape, lens, [1] * 7, "decode", splits, uniform=splits == 2) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("shape", SHAPES)
def test_latent_decode_takes_ragged_portions(shape):
    assert _latent_case(torch.bfloat16, *shape, [5, 130, 257, 9, 64], [5, 1, 7, 2, 16], "decode", 2) < OP_TOL[torch.bfloat16]
    assert _latent_case(torch.bfloat16, *shape, [130, 66], [3, 3], "decode", 3, bs=32, uniform=True) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("shape", [s for s in SHAPES if s[2] <= 64])
def test_latent_prefill(shape):
    lens = [401, 1, 130, 257, 37]
    assert _latent_case(torch.bfloat16, *shape, lens, lens, "fresh") < OP_TOL[torch.bfloat16]
    q_lens = [150, 1, 2, 257, 20]
    assert _latent_case(torch.bfloat16, *shape, lens, q_lens, "context") < OP_TOL[torch.bfloat16]
    assert _latent_case(torch.bfloat16, *shape, lens, q_lens, "context", listed=[3, 0, 4]) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [SHAPES[1], (2, 136, 72, 132, 600), (1, 10, 2, 9, 900)])
def test_latent_attention_outside_the_tensor_core_kernels(dtype, shape):
    assert _latent_case(dtype, *shape, [100, 3, 75], [60, 2, 1], "simple") < OP_TOL[dtype]
    assert _latent_case(dtype, *shape, [100, 75], [1, 1], "simple", scale=-0.1, uniform=True) < OP_TOL[dtype]


@pytest.mark.parametrize("plant", [0, 1, 15, 16, 63, 64, 127, 128, -2, -1])
@pytest.mark.parametrize("how", ["fresh", "context", "decode", "simple"])
def test_far_keys_and_page_borders_carry_the_weight(plant, how):
    """One key that takes the whole softmax of the last query, far away, at page and tile borders, and the query's own."""
    lens = [385, 130, 64]
    q_lens = lens if how == "fresh" else [40, 1, 17] if how == "context" else [1, 2, 1]
    for dtype in DTYPES if how == "simple" else DTYPES[1:]:
        assert _latent_case(dtype, 4, 48, 16, 32, 64, lens, q_lens, how, 2, plant=plant) < OP_TOL[dtype]


@pytest.mark.parametrize("mean", [-40.0, 6.0, 60.0])
@pytest.mark.parametrize("how,splits", [("fresh", 1), ("context", 1), ("decode", 1), ("decode", 4)])
def test_sinks_of_any_size(mean, how, splits):
    lens = [200, 130]
    q_lens = [1, 1] if how == "decode" else lens if how == "fresh" else [50, 2]
    assert _latent_case(torch.bfloat16, 4, 64, 16, 64, 128, lens, q_lens, how, splits, sink_mean=mean) < OP_TOL[torch.bfloat16]


# ---- delta rule -----------------------------------------------------------------------------------------------------------
def _delta_inputs(dtype, H, G, D, E, taps, T, seed=0, slow=False):
    """(DeltaWeights, plain tensors, projections [T, cols] with padding, decay and gate logits)."""
    from inference_b200 import ops

    dp, vp, up8 = ops.delta_key_width(D), (E + 7) // 8 * 8, lambda n: (n + 7) // 8 * 8
    x = {n: rnd(T, h, d, seed=seed + i, dtype=torch.bfloat16).float() for i, (n, h, d) in enumerate((("q", G, D), ("k", G, D), ("v", H, E)))}
    cw = {n: rnd(x[n].shape[1] * x[n].shape[2], taps, seed=seed + 5 + i, std=taps ** -0.5, dtype=torch.bfloat16).float() for i, n in enumerate("qkv")}
    b, dl, gl = (rnd(T, *s, seed=seed + 9 + i, dtype=torch.bfloat16).float() for i, s in enumerate(((H,), (H, D), (H, E))))
    a_log = rnd(H, seed=seed + 13) * 0.5 - (6.0 if slow else 2.0)
    dt, norm = rnd(H, D, seed=seed + 14) - 1.0, 1 + 0.3 * rnd(E, seed=seed + 15)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))   # noqa: E731
    widths = {"q": dp, "k": dp, "v": vp}
    col_b = 2 * G * dp + H * vp
    proj = torch.cat([pad(x[n], widths[n]).reshape(T, -1) for n in "qkv"] + [pad(b, up8(H))], 1)
    conv = torch.cat([torch.nn.functional.pad(cw[n].view(*x[n].shape[1:], taps), (0, 0, 0, widths[n] - x[n].shape[2])).reshape(-1, taps)
                      for n in "qkv"]).t().contiguous()
    w = ops.DeltaWeights(H, G, D, dp, E, vp, col_b, conv.cuda(), a_log.cuda(), pad(dt, dp).reshape(-1).cuda(), pad(norm, vp).cuda())
    plain = dict(x=x, cw=cw, b=b, dl=dl, gl=gl, a_log=a_log, dt=dt, norm=norm)
    return w, plain, proj.to(dtype), pad(dl, dp).reshape(T, -1).to(dtype), pad(gl, vp).reshape(T, -1).to(dtype)


def _delta_want(p, lo, hi, H, eps):
    """Rows lo..hi of the flat batch as one sequence of its own."""
    s = slice(lo, hi)
    conv = {n: ref.causal_conv_silu(p["x"][n][s].double().flatten(1), p["cw"][n].double()).view(p["x"][n][s].shape) for n in "qkv"}
    D = conv["q"].shape[2]
    g = ref.decay(p["dl"][s].double().flatten(1), p["a_log"].double(), p["dt"].double().flatten(), H)
    o, S = ref.delta_rule(ref.unit(conv["q"]) * D ** -0.5, ref.unit(conv["k"]), conv["v"], g, torch.sigmoid(p["b"][s].double()))
    return ref.rms(o, eps) * p["norm"].double() * torch.sigmoid(p["gl"][s].double()), S


DELTA = [(6, 3, 24, 40, 4), (2, 2, 32, 64, 4), (2, 1, 10, 12, 2), (1, 1, 33, 7, 5), (4, 2, 64, 8, 3), (3, 3, 90, 100, 4), (4, 4, 128, 128, 4),
         (2, 1, 140, 72, 1), (2, 2, 200, 24, 4), (2, 1, 300, 40, 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", DELTA)
def test_delta_rule_over_portions(dtype, shape):
    """Three sequences cut differently: whole, in portions down to one and two tokens, token by token; states and windows carry
    over, slots that no sequence owns stay as they are."""
    from inference_b200 import ops

    H, G, D, E, taps = shape
    lens, eps = [70, 41, 9], 1e-3
    starts = [0, 70, 111]
    w, p, proj, dec, gate = _delta_inputs(dtype, H, G, D, E, taps, sum(lens))
    state, window = torch.full((5, *w.state_shape()), 3.0, device="cuda"), torch.full((5, *w.window_shape()), 3.0, device="cuda", dtype=dtype)
    slot, at = [3, 0, 2], [0, 0, 0]
    got = torch.zeros(sum(lens), H, w.vp)
    plan = [(70, 1, 2), (0, 2, 1), (0, 16, 1), (0, 1, 1), (0, 3, 1), (0, 17, 1), (0, 1, 2)]
    for cut in plan:
        live = [i for i in range(3) if cut[i]]
        idx = torch.cat([torch.arange(starts[i] + at[i], starts[i] + at[i] + cut[i]) for i in live])
        pos = torch.cat([torch.arange(at[i], at[i] + cut[i]) for i in live]).int().cuda()
        cu = i32([0] + [cut[i] for i in live]).cumsum(0).int()
        out = ops.channel_delta(proj[idx].cuda(), dec[idx].cuda(), gate[idx].cuda(), w, eps, state, window, i32([slot[i] for i in live]), pos,
                                cu_q=cu, max_q_len=max(cut))
        got[idx] = out.view(-1, H, w.vp).float().cpu()
        for i in live:
            at[i] += cut[i]
    assert at == lens
    for i in range(3):
        want, S = _delta_want(p, starts[i], starts[i] + lens[i], H, eps)
        assert rel(got[starts[i]:starts[i] + lens[i], :, :E], want) < OP_TOL[dtype]
        assert rel(state[slot[i], :, :E, :D].transpose(1, 2), S) < (1e-5 if dtype == torch.float32 else 3e-3)
    assert (state[[1, 4]] == 3).all() and (window[[1, 4]] == 3).all() and (got[..., E:] == 0).all()


def test_delta_rule_slot_reuse_and_padding_rows():
    """A slot that is used again starts from zero at position 0; rows with slot -1 (padding of a decode batch) touch nothing."""
    from inference_b200 import ops

    H, G, D, E, taps = 4, 2, 32, 24, 4
    w, p, proj, dec, gate = _delta_inputs(torch.float32, H, G, D, E, taps, 12)
    state, window = torch.full((2, *w.state_shape()), float("nan"), device="cuda"), torch.full((2, *w.window_shape()), float("nan"), device="cuda")
    run = lambda lo, hi, slots, pos: ops.channel_delta(proj[lo:hi].cuda(), dec[lo:hi].cuda(), gate[lo:hi].cuda(), w, 1e-5, state, window,   # noqa: E731
                                                       i32(slots), i32(pos), cu_q=None, max_q_len=(hi - lo) // len(slots))
    run(0, 3, [1], [0, 1, 2])
    out = torch.cat([run(3, 11, [1], list(range(8))), run(11, 12, [1], [8])])
    assert rel(out.view(9, H, -1)[..., :E], _delta_want(p, 3, 12, H, 1e-5)[0]) < 1e-5
    keep = state.clone(), window.clone()
    run(0, 3, [-1, -1, -1], [5, 5, 5])
    assert torch.equal(state[1], keep[0][1]) and torch.equal(window[1], keep[1][1]) and state[0].isnan().all()


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_remembers_far_tokens(dtype):
    """Slow decays: what the first tokens wrote is still read 900 tokens later, in fp32 state."""
    from inference_b200 import ops

    H, G, D, E, T = 2, 1, 32, 16, 900
    w, p, proj, dec, gate = _delta_inputs(dtype, H, G, D, E, 4, T, slow=True)
    for t in (proj, p["b"]):                                     # nearly no writes after the first ten tokens
        t[10:, w.col_b if t is proj else 0:][:, :H] = -9.0
    state, window = torch.zeros((1, *w.state_shape()), device="cuda"), torch.zeros((1, *w.window_shape()), device="cuda", dtype=dtype)
    got, at = [], 0
    for n in (500, 37, 300, 62, 1):
        got.append(ops.channel_delta(proj[at:at + n].cuda(), dec[at:at + n].cuda(), gate[at:at + n].cuda(), w, 1e-5, state, window, i32([0]),
                                     torch.arange(at, at + n, device="cuda").int(), cu_q=None, max_q_len=n))
        at += n
    want, S = _delta_want(p, 0, T, H, 1e-5)
    first, _ = _delta_want({**p, "b": torch.cat([torch.full((10, H), -40.0), p["b"][10:]])}, 0, T, H, 1e-5)
    got = torch.cat(got).view(T, H, -1)[..., :E]
    assert rel(got[-60:], want[-60:]) < OP_TOL[dtype] and rel(first[-60:], want[-60:]) > 0.3


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


def _idle(backend):
    pool = backend.runner.pool
    return pool.allocator.live_blocks() == 0 and (pool.slots is None or pool.slots.live_blocks() == 0)


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
    worst = max(rel(g, w) for g, w in zip(got, want))
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
def test_mixed_batches_reused_pages_and_slots(dtype):
    """Portions of some sequences beside single tokens of others, sequences that pause, end and give their pages and state slots
    to new ones; both are just enough. Every logit equals that of the sequence alone."""
    lens = {"p": 90, "q": 33, "r": 150, "s": 17, "t": 120, "u": 64}
    toks = {k: _tokens("a", n, 10 + i) for i, (k, n) in enumerate(lens.items())}
    b = _backend("a", dtype, max_batch=4, ctx=160, kv_tokens=352)
    assert b.runner.pool.slots.capacity == 4
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
@pytest.mark.parametrize("name", ["a", "e"])
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
    """19 rows decode in a graph captured for 24: the padding rows own no state and write nothing, and capturing advances none."""
    b = _backend("b", dtype, max_batch=24, ctx=64, kv_tokens=24 * 64)
    toks = [_tokens("b", 12 + i, 100 + i) for i in range(19)]
    seqs = [b.new_sequence() for _ in toks]
    b.forward_at(seqs, [t[:-3] for t in toks], [[] for _ in toks])
    for back in (3, 2, 1):
        got = b.forward_at(seqs, [[t[-back]] for t in toks], [[0] for _ in toks])
        for g, t in zip(got, toks):
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
    assert llm.descriptor().family == "gunedra"
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
