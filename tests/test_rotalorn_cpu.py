"""Rotalorn host side without a GPU: config reading, registry, weight checks and padding, cache geometry, token pages under forks and
rollbacks, KV splits, the division of a step, and whether the test models show mistakes."""
import copy
import json

import pytest
import torch

import rotalorn_reference as ref


def _cfg(name="a"):
    from inference_b200.models import ModelConfig

    return ModelConfig.from_json(ref.MODELS[name]())


def test_config_reads_every_size_and_constant():
    from inference_b200.models import Architecture
    from inference_b200.models.config import (AttentionSpec, BigramSpec, DenseSpec, DifferentialSpec, ExpertsSpec, LatentAttentionSpec,
                                              RopeScaling)

    c = _cfg()
    assert c.architecture is Architecture.ROTALORN and (c.hidden_size, c.vocab_size, c.rms_norm_eps) == (144, 311, 1e-3)
    s = c.stack
    assert s.bigram == BigramSpec(97, 13, 29) and s.loop is None and s.logit_scale == 1.0
    assert s.layers[0].mixer == AttentionSpec(6, 2, 40, 40, 40 ** -0.5, 0, 24, 700.0, RopeScaling(8.0, 1.0, 4.0, 96.0), 24)
    assert s.layers[0].mlp == ExpertsSpec(6, 3, 24, 40)
    assert s.layers[1].mixer == DifferentialSpec(4, 2, 24, 40, 24 ** -0.5, 15.0, 0.35, 0.3, 16.0) and s.layers[1].mlp == DenseSpec(120)
    assert s.layers[2].mixer == LatentAttentionSpec(5, 24, 8, 40, 48, 32 ** -0.5, 900.0, 72, 33)
    assert s.layers[3].mlp is None and s.layers[4].mixer.rot_scaling is None and s.layers[4].mixer.scale == 0.3
    assert c.to_json() == ref.model_a() and c.groups == 5


@pytest.mark.parametrize("path,value", [(("width",), None), (("vocab",), 0), (("norm", "eps"), None), (("embedding",), None),
                                        (("embedding", "bigram"), None), (("embedding", "bigram", "buckets"), 0),
                                        (("embedding", "bigram", "mul_cur"), None), (("layers", 0, "mixer", "scale"), None),
                                        (("layers", 0, "mixer", "kv_heads"), 4), (("layers", 0, "mixer", "vdim"), 32),
                                        (("layers", 0, "mixer", "rot", "dims"), 25), (("layers", 0, "mixer", "mask", "size"), 0),
                                        (("layers", 0, "mixer", "rot", "scaling", "original"), None), (("layers", 0, "mlp", "router", "top"), 7),
                                        (("layers", 0, "mlp", "shared"), None), (("layers", 1, "mixer", "diff"), None),
                                        (("layers", 1, "mixer", "softcap"), -1), (("layers", 1, "mixer", "q_temp", "every"), 0),
                                        (("layers", 1, "mixer", "q_temp", "coef"), None), (("layers", 1, "mlp", "ff"), None),
                                        (("layers", 2, "mixer", "q_rank"), None), (("layers", 2, "mixer", "rot", "dims"), 6), (("layers",), [])])
def test_config_errors_name_the_key(path, value):
    from inference_b200.contracts.errors import ConfigError
    from inference_b200.models import ModelConfig

    j = copy.deepcopy(ref.model_a())
    d = j
    for p in path[:-1]:
        d = d[p]
    d[path[-1]] = value
    with pytest.raises(ConfigError):
        ModelConfig.from_json(j)


def test_parts_of_other_designs_are_refused():
    from inference_b200.contracts.errors import Unsupported
    from inference_b200.models import ModelConfig

    for edit in (lambda j: j["layers"][0].update(type="channel_delta"), lambda j: j["layers"][1]["mlp"].update(kind="sparse"),
                 lambda j: j.update(architecture="Rotalor")):
        j = copy.deepcopy(ref.model_a())
        edit(j)
        with pytest.raises(Unsupported):
            ModelConfig.from_json(j)


def test_registry_and_providers(tmp_path):
    from inference_b200.contracts.core_llm import LoadSpec
    from inference_b200.engine.provider import B200_LLAMA, CPU_LLAMA
    from inference_b200.models.registry import gpu_model, gpu_supported
    from inference_b200.models.rotalorn import RotalornGpu

    m = gpu_model(_cfg(), device=torch.device("cpu"))
    assert gpu_supported(_cfg()) and isinstance(m, RotalornGpu) and not m.recurrent
    (tmp_path / "config.json").write_text(json.dumps(ref.model_a()))
    spec = LoadSpec.dense(str(tmp_path))
    assert B200_LLAMA.can_load(spec) and not CPU_LLAMA.can_load(spec)


@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_weights_land_padded_and_complete(name):
    """Every projection, applied by hand to padded inputs in the order of the padded layouts, equals the plain one."""
    from inference_b200.models.latent_mixer import half_pairs
    from inference_b200.models.rotalorn import RotalornGpu

    cfg, w = ref.MODELS[name](), ref.random_weights(ref.MODELS[name]())
    m = RotalornGpu(_cfg(name), device=torch.device("cpu"), dtype=torch.float32).load_state_dict(w)
    W = cfg["width"]
    Wt = {k: t.float() for k, t in w.items()}
    x = torch.randn(3, W)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))   # noqa: E731
    xp = pad(x, m.hp)
    same = lambda a, b: torch.allclose(a, b, atol=2e-4)   # noqa: E731
    assert torch.equal(m.pairs[:, :W], Wt["bigram"]) and torch.equal(m.embed[:, :W], Wt["embed"]) and torch.equal(m.final.b[:W], Wt["final.norm.b"])
    for i, (lay, spec) in enumerate(zip(m.layers, cfg["layers"])):
        s, p, f = spec["mixer"], f"l{i}.mix.", spec["mlp"]
        H, E = s["heads"], s["vdim"]
        proj = xp @ lay.w_in.T + (lay.b_in if lay.b_in is not None else 0)
        assert torch.equal(lay.norm.w[:W], Wt[f"l{i}.norm1"]) and torch.equal(lay.norm.b[:W], Wt[f"l{i}.norm1.b"]) and (lay.norm.b[W:] == 0).all()
        vorder = list(range(E))
        if spec["type"] == "attention":
            G, D = s["kv_heads"], s["dim"]
            vorder = order = half_pairs(D, s["rot"]["dims"])
            for n, h, t in (("q", H, proj[:, :H * lay.dk]), ("k", G, proj[:, H * lay.dk:])):
                t = t.reshape(3, h, lay.dk)
                assert same(t[..., :D], (x @ Wt[p + n].T + Wt[f"{p}{n}.b"]).view(3, h, D)[..., order]) and (t[..., D:] == 0).all()
                got = (lay.q_norm if n == "q" else lay.k_norm).view(h, lay.dk)
                assert torch.equal(got[:, :D], Wt[f"{p}{n}.norm"].view(h, D)[:, order]) and (got[:, D:] == 0).all()
        elif spec["type"] == "attention_2":
            G, D = s["kv_heads"], s["dim"]
            q, k, v = proj.split([H * 2 * lay.dk, G * 2 * lay.dk, G * lay.dv], 1)
            for n, t, h, d, dp in (("q", q, 2 * H, D, lay.dk), ("k", k, 2 * G, D, lay.dk), ("v", v, G, E, lay.dv)):
                t = t.reshape(3, h, dp)
                assert same(t[..., :d].reshape(3, -1), x @ Wt[p + n].T) and (t[..., d:] == 0).all()
            assert abs(lay.share - float(ref.second_map_share({k: t.double() for k, t in w.items()}, p, s["diff"]))) < 1e-9
        else:
            z = lay.latent
            order = half_pairs(s["rot_dim"], s["rot_dim"])
            assert z.window == s["mask"]["size"] and z.sink is None
            assert same(proj[:, :z.q_rank], x @ Wt[p + "dq"].T) and (proj[:, z.q_rank:z.qk] == 0).all()
            low = x @ Wt[p + "dkv"].T
            assert same(proj[:, z.col_c:z.col_c + z.rank], low[:, :z.rank])
            assert same(proj[:, z.col_c + z.rk:z.col_c + z.rk + z.rot], low[:, z.rank:][:, order])
            assert same(proj[:, z.col_gate:z.col_gate + H], x @ Wt[p + "g"].T)
            c = torch.randn(3, z.q_rank)
            q = (pad(c, z.qk) @ z.uq.T).view(3, H, z.dn + z.rp)
            want = (c @ Wt[p + "uq"].T).view(3, H, -1)
            assert same(q[..., :z.dim], want[..., :z.dim]) and same(q[..., z.dn:z.dn + z.rot], want[..., z.dim:][..., order])
            c = torch.randn(3, z.rank)
            assert same((pad(c, z.rk) @ z.uv.transpose(1, 2)).transpose(0, 1)[..., :E].reshape(3, -1), c @ Wt[p + "uv"].T)
        a, want = torch.randn(3, H, E), 0
        cat = [pad(a[..., vorder], lay.dv).reshape(3, -1)]
        if f is not None:
            q = f"l{i}.mlp." + ("shared." if f["kind"] == "moe" else "")
            ff = Wt[q + "gate"].shape[0]
            u = torch.randn(3, ff)
            cat.append(pad(u, (ff + 7) // 8 * 8))
            want = u @ Wt[q + "down"].T
            gu = (xp @ lay.ff.gate_up.T).view(3, -1, 2)[:, :ff]
            assert same(gu[..., 0], x @ Wt[q + "gate"].T) and same(gu[..., 1], x @ Wt[q + "up"].T)
            if f["kind"] == "moe":
                n = f["router"]["experts"]
                z = xp @ lay.ff.router.T
                assert same(z[:, :n], x @ Wt[f"l{i}.mlp.router"].T) and same(z[:, n:n + 1], x @ Wt[q + "sg"].T)
                e = n - 1
                gu = (xp @ lay.ff.experts_in[e].T).view(3, -1, 2)[:, :f["expert"]["ff"]]
                u = torch.randn(3, f["expert"]["ff"])
                assert same(gu[..., 1], x @ Wt[f"l{i}.mlp.e{e}.up"].T)
                assert same((pad(u, lay.ff.experts_out.shape[2]) @ lay.ff.experts_out[e].T)[:, :W], u @ Wt[f"l{i}.mlp.e{e}.down"].T)
        y = torch.cat(cat, 1) @ lay.w_out.T
        assert same(y[:, :W], a.reshape(3, -1) @ Wt[p + "o"].T + want) and (y[:, W:] == 0).all()


def test_weight_errors():
    from inference_b200.contracts.errors import LoadError, Unsupported
    from inference_b200.models import ModelConfig
    from inference_b200.models.rotalorn import RotalornGpu

    def load(w):
        return RotalornGpu(_cfg(), device=torch.device("cpu")).load_state_dict(w)
    good = ref.random_weights(ref.model_a())
    load(good)
    for name, t in (("l0.mix.q.b", None), ("l0.mix.k.norm", torch.zeros(40)), ("bigram", torch.zeros(97, 144)), ("l0.mlp.e5.up", None),
                    ("l0.mlp.shared.sg", torch.zeros(144)), ("l1.mix.lq2", None), ("l2.mix.uq", torch.zeros(160, 71)), ("l3.norm1.b", None)):
        w = dict(good)
        if t is None:
            del w[name]
        else:
            w[name] = t
        with pytest.raises(LoadError):
            load(w)
    j = ref.model_a()
    j["layers"][1]["mixer"]["dim"] = 1025
    with pytest.raises(Unsupported):
        RotalornGpu(ModelConfig.from_json(j), device=torch.device("cpu"))


def test_pool_pages_tokens_beside_keys():
    from inference_b200.engine.kv_pool import LayeredKvPool, PagedSequence
    from inference_b200.models.registry import gpu_model

    m = gpu_model(_cfg(), device=torch.device("cpu"))
    pool = m.make_pool(6, 4)
    shapes = [[tuple(t.shape) for t in kv] for kv in pool.data]
    assert shapes == [[(6, 2, 4, 40), (6, 2, 4, 40)], [(6, 2, 4, 48), (6, 2, 4, 40)], [(6, 4, 128)], [(6, 3, 4, 128), (6, 3, 4, 128)],
                      [(6, 4, 4, 24), (6, 4, 4, 24)], [(6, 4)]]
    assert pool.data[-1][0].dtype == torch.int32 and pool.data[0][0].dtype == torch.bfloat16 and not pool.has_state
    per_token = 2 * (160 + 96 + 80 + 128 + 768 + 192) + 4
    assert m.kv_block_bytes(4) == 4 * per_token == LayeredKvPool.block_bytes(m.kv_geometry(), 4, 2)
    # a fork shares whole pages; what it writes behind them lands in pages of its own, token ids included
    s = PagedSequence(pool)
    for slot, t in zip(s.reserve(6), range(10, 16)):
        pool.data[-1][0].view(-1)[slot] = t
    f = PagedSequence.seeded(pool, list(s.blocks), 6)
    slot = f.reserve(1)[0]
    pool.data[-1][0].view(-1)[slot] = 99
    ids = lambda q: [int(pool.data[-1][0][q.blocks[i // 4], i % 4]) for i in range(q.length)]   # noqa: E731
    assert ids(s) == list(range(10, 16)) and ids(f) == [*range(10, 16), 99] and f.blocks[0] == s.blocks[0] and f.blocks[1] != s.blocks[1]
    f.truncate(5)
    assert ids(f) == list(range(10, 15))
    for q in (s, f):
        q.release()
    assert pool.allocator.live_blocks() == 0


def test_splits_follow_the_windows():
    from inference_b200.models.registry import gpu_model

    m = gpu_model(_cfg("d"), device=torch.device("cpu"))
    long, short = m.decode_splits(1, 100000), m.decode_splits(1, 1)
    assert long[0] == 32 and long[1] == m.decode_splits(1, 263)[1] == 2 and long[2] == m.decode_splits(1, 192)[2] <= 4 and short == (1, 1, 1)
    assert m.decode_splits(500, 5000) == (1, 1, 1)


def test_a_step_gathers_only_the_keys_of_its_windows():
    from inference_b200.models.latent_mixer import Ragged
    from inference_b200.models.llama import StepInputs
    from inference_b200.models.registry import gpu_model

    r = Ragged(3, 0, 0, 0, spans=[(20, 100), (30, 30), (17, 40)])
    cpu = torch.device("cpu")
    cu, first, n = r.keys(33, cpu)
    assert cu.tolist() == [0, 52, 82, 122] and first.tolist() == [48, 0, 0] and n == 122
    cu, first, n = r.keys(0, cpu)
    assert cu.tolist() == [0, 100, 130, 170] and first is None and n == 170
    m = gpu_model(_cfg(), device=cpu)
    z = torch.zeros(38, dtype=torch.int64)
    inp = StepInputs(input_ids=z, positions=z.int(), slot_mapping=z, block_table=z.view(2, 19).int(), kv_lens=torch.tensor([9, 30, 60]).int(),
                     cu_q=torch.tensor([0, 1, 21, 38]).int(), max_q_len=20, num_seqs=3, decode=False, spans=[(1, 9), (20, 30), (17, 60)])
    few, many = m._split_step(inp)
    assert few.rows.tolist() == [0] and few.cu.tolist() == [0, 1] and few.q_row.tolist() == [0] + [-1] * 37
    assert many.seqs.tolist() == [1, 2] and many.spans == [(20, 30), (17, 60)] and many.keys(33, cpu)[1].tolist() == [0, 11]


def _edit(path, fn):
    def go(cfg, w):
        for lay in cfg["layers"]:
            d = lay
            for p in path[:-1]:
                d = d.get(p) or {}
            if path[-1] in d:
                d[path[-1]] = fn(d[path[-1]])
        return cfg, w
    return go


def _change(suffix, fn):
    return lambda cfg, w: (cfg, {k: (fn(t) if k.endswith(suffix) else t) for k, t in w.items()})


def _pairs(**kw):
    def go(cfg, w):
        cfg["embedding"]["bigram"].update(kw)
        return cfg, w
    return go


def _drop_scaling(cfg, w):
    for lay in cfg["layers"]:
        (lay["mixer"].get("rot") or {}).pop("scaling", None)
    return cfg, w


@pytest.mark.parametrize("mistake", [_pairs(mul_prev=14), _pairs(mul_cur=28), _drop_scaling, _edit(("mixer", "rot", "base"), lambda b: b * 1.5),
                                     _edit(("mixer", "mask", "size"), lambda n: n - 1), _edit(("mixer", "mask", "size"), lambda n: n + 1),
                                     _edit(("mixer", "scale"), lambda s: s * 1.3), _edit(("mixer", "softcap"), lambda c: c * 0.3),
                                     _edit(("mixer", "diff"), lambda d: d * 0.7), _edit(("mixer", "q_temp", "coef"), lambda c: 0.0),
                                     _edit(("mixer", "q_temp", "every"), lambda n: n * 2), _edit(("mlp", "router", "top"), lambda n: n - 1),
                                     _change("q.b", torch.zeros_like), _change("k.b", torch.zeros_like), _change(".q.norm", lambda t: t.roll(1)),
                                     _change(".k.norm", lambda t: t.roll(1)), _change("dq.norm", lambda t: t.roll(1)),
                                     _change("dkv.norm", lambda t: t.roll(1)), _change("mix.g", torch.zeros_like), _change(".sg", torch.zeros_like),
                                     _change(".lq1", torch.zeros_like), _change(".lk2", torch.zeros_like), _change("norm1.b", torch.zeros_like),
                                     _change("router", lambda t: t.roll(1, 0))])
def test_test_models_are_sensitive_to_mistakes(mistake):
    """A mistake planted in the restatement moves the logits of the test models far beyond the tolerances of the GPU tests in 32-bit, and
    beyond those in bf16 for some positions."""
    tokens = torch.randint(0, 311, (60,), generator=torch.Generator().manual_seed(2)).tolist()
    cfg, w = ref.model_a(), ref.random_weights(ref.model_a(), seed=ord("a"))
    good = ref.run(cfg, w, tokens)[0]
    bad = ref.run(*mistake(copy.deepcopy(cfg), w), tokens)[0]
    err = (good - bad).square().mean(-1).sqrt() / good.square().mean(-1).sqrt()
    assert float(err.square().mean().sqrt()) > 0.02 and float(err.max()) > 0.05


def test_restatement_pieces():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)   # noqa: E731
    assert ref.bigram_rows([5, 3, 9], 10, 3, 7) == [10, (15 + 21) % 10, (9 + 63) % 10]
    n = ref.layer_norm(r(4, 30) * 3 + 2, torch.ones(30, dtype=torch.float64), torch.zeros(30, dtype=torch.float64), 0.0)
    assert torch.allclose(n.mean(-1), torch.zeros(4, dtype=torch.float64), atol=1e-12) and torch.allclose(n.square().mean(-1), torch.ones(4, dtype=torch.float64))
    # rotation by halves: dimension 0 pairs with dims / 2, the rest stay
    x = torch.zeros(1, 1, 6, dtype=torch.float64)
    x[0, 0, 0], x[0, 0, 5] = 1.0, 7.0
    y = ref.rotate_halves(x, torch.tensor([2]), {"dims": 4, "base": 100.0})[0, 0]
    a = torch.tensor(2.0, dtype=torch.float64)
    assert torch.allclose(y, torch.stack([a.cos(), 0 * a, a.sin(), 0 * a, 0 * a, 7 + 0 * a]))
    ok = ref.visible(torch.tensor([5]), 8, 3)
    assert ok[0].tolist() == [False, False, False, True, True, True, False, False]
    assert torch.allclose(ref.temperature(torch.tensor([0, 6, 7, 15]), 0.5, 8), 1 + 0.5 * torch.log(torch.tensor([1.0, 1.0, 2.0, 3.0], dtype=torch.float64)))
    k, v = r(5, 1, 4), r(5, 1, 3)
    one = ref.softmax_attention(r(1, 1, 4), k, v, torch.tensor([3]), 0.5, 1)
    assert torch.allclose(one[0, 0], v[3, 0])
    e, s = ref.route(r(3, 6), r(4, 6), 4)
    assert torch.allclose(s.sum(-1), torch.ones(3, dtype=torch.float64)) and ref.margin(r(3, 6), r(4, 6), 4).isinf().all()
