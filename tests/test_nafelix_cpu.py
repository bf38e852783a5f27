"""Nafelix host side without a GPU: config reading, registry, weight checks and padding, cache and state geometry, KV splits, the exchange
of weights behind the values, and whether the test models show mistakes."""
import copy
import json

import pytest
import torch

import nafelix_reference as ref


def _cfg(name="a"):
    from inference_b200.models import ModelConfig

    return ModelConfig.from_json(ref.MODELS[name]())


def test_config_reads_every_size_and_constant():
    from inference_b200.models import Architecture
    from inference_b200.models.config import AttentionSpec, DenseSpec, ExpertsSpec, HeadDeltaSpec, LoopSpec, ParallelSpec

    c = _cfg()
    assert c.architecture is Architecture.NAFELIX and (c.hidden_size, c.vocab_size, c.rms_norm_eps) == (144, 311, 1e-3)
    s = c.stack
    assert (s.streams, s.canon_taps, s.loop, s.tied) == (4, 4, LoopSpec(1, 3, 3), False) and not c.tie_word_embeddings
    assert s.layers[0].mixer == ParallelSpec(AttentionSpec(6, 3, 40, 24, 40 ** -0.5, 0, 24, 700.0, None, 24), HeadDeltaSpec(6, 2, 24, 40, 3))
    assert s.layers[0].mlp == ExpertsSpec(4, 4, 24, limit=0.8) and s.layers[1].mlp is None and s.layers[2].mlp == DenseSpec(120)
    assert s.layers[1].mixer == AttentionSpec(6, 2, 24, 56, 24 ** -0.5, 0, 8, 500.0, None, 33) and s.layers[2].mixer.left.scale == 0.3
    assert c.to_json() == ref.model_a() and c.groups == 4
    assert [i for i, _ in s.runs()] == [0, 1, 2, 1, 2, 1, 2, 3] == ref.runs(ref.model_a())
    j = ref.model_a()
    j["loop"] = None
    del j["layers"][1]["mixer"]["mask"], j["layers"][1]["mixer"]["rot"]
    from inference_b200.models import ModelConfig
    c = ModelConfig.from_json(j)
    assert c.stack.loop is None and c.stack.layers[1].mixer.window == 0 and c.stack.layers[1].mixer.rot_dims == 0


@pytest.mark.parametrize("path,value", [(("width",), None), (("vocab",), 0), (("norm", "eps"), None), (("streams",), None), (("streams",), 0),
                                        (("canon",), None), (("canon", "taps"), 0), (("loop", "stop"), 9), (("loop", "times"), 0),
                                        (("layers", 0, "mixer", "left"), None), (("layers", 0, "mixer", "right"), None),
                                        (("layers", 0, "mixer", "left", "kv_heads"), 4), (("layers", 0, "mixer", "left", "scale"), None),
                                        (("layers", 0, "mixer", "left", "rot", "dims"), 25), (("layers", 0, "mixer", "left", "mask", "size"), 0),
                                        (("layers", 0, "mixer", "right", "conv"), None), (("layers", 0, "mixer", "right", "kv_heads"), 4),
                                        (("layers", 0, "mlp", "router", "top"), 5), (("layers", 0, "mlp", "expert", "limit"), None),
                                        (("layers", 0, "mlp", "expert", "limit"), -1), (("layers", 1, "mixer", "rot", "base"), None),
                                        (("layers", 1, "mixer", "rot", "dims"), 26), (("layers", 2, "mlp", "ff"), None), (("layers",), [])])
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

    for edit in (lambda j: j["layers"][0].update(type="channel_delta"), lambda j: j["layers"][2]["mlp"].update(kind="gated"),
                 lambda j: j.update(architecture="Nafeli")):
        j = copy.deepcopy(ref.model_a())
        edit(j)
        with pytest.raises(Unsupported):
            ModelConfig.from_json(j)


def test_registry_and_providers(tmp_path):
    from inference_b200.contracts.core_llm import LoadSpec
    from inference_b200.engine.provider import B200_LLAMA, CPU_LLAMA
    from inference_b200.models.nafelix import NafelixGpu
    from inference_b200.models.registry import gpu_model, gpu_supported

    m = gpu_model(_cfg(), device=torch.device("cpu"))
    assert gpu_supported(_cfg()) and isinstance(m, NafelixGpu) and m.recurrent
    (tmp_path / "config.json").write_text(json.dumps(ref.model_a()))
    spec = LoadSpec.dense(str(tmp_path))
    assert B200_LLAMA.can_load(spec) and not CPU_LLAMA.can_load(spec)


def test_values_share_a_tile():
    from inference_b200.models.nafelix import values_together

    assert [values_together(*a) for a in ((2, 32), (4, 64), (3, 64), (6, 24), (8, 128), (1, 200), (12, 8), (4, 32))] == [2, 2, 1, 3, 1, 1, 12, 4]


@pytest.mark.parametrize("name", list(ref.MODELS))
def test_weights_land_padded_and_complete(name):
    """Every projection, applied by hand to padded inputs in the order of the padded layouts, equals the plain one."""
    from inference_b200.models.nafelix import NafelixGpu
    from inference_b200.models.stack import half_pairs

    cfg, w = ref.MODELS[name](), ref.random_weights(ref.MODELS[name]())
    m = NafelixGpu(_cfg(name), device=torch.device("cpu"), dtype=torch.float32).load_state_dict(w)
    W = cfg["width"]
    Wt = {k: t.float() for k, t in w.items()}
    x = torch.randn(3, W)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))   # noqa: E731
    xp, up8 = pad(x, m.hp), lambda n: (n + 7) // 8 * 8                     # noqa: E731
    same = lambda a, b: torch.allclose(a, b, atol=2e-4)                   # noqa: E731
    assert torch.equal(m.embed[:, :W], Wt["embed"]) and torch.equal(m.head[:, :W], Wt["head"]) and torch.equal(m.final.w[:W], Wt["final.norm"])

    def check_attention(a, s, p, proj, gate_rows):
        H, G, D, E = s["heads"], s["kv_heads"], s["dim"], s["vdim"]
        order, vp = half_pairs(D, s["rot"]["dims"]), up8(E)
        q, k, v, gate = proj.split([*a.cols, gate_rows], 1)
        for n, t, h, d, dp, o in (("q", q, H, D, a.dk, order), ("k", k, G, D, a.dk, order), ("v", v, G, E, vp, list(range(E)))):
            t = t.reshape(3, h, dp)
            want = x @ Wt[p + n].T + Wt.get(f"{p}{n}.b", 0)
            assert same(t[..., :d], want.view(3, h, d)[..., o]) and (t[..., d:] == 0).all()
        z = torch.randn(3, H, E)
        y = pad(z, vp).reshape(3, -1) @ a.o.T
        assert same(y[:, :W], z.reshape(3, -1) @ Wt[p + "o"].T) and (y[:, W:] == 0).all()
        assert torch.equal(a.sink, Wt[p + "sink"]) and a.value_heads * a.dv == G * vp
        return gate

    def check_sublayer(sub, L, n):
        assert torch.equal(sub.norm.w[:W], Wt[f"{L}norm{n}"]) and (sub.norm.w[W:] == 0).all()
        assert torch.equal(sub.read, Wt[f"{L}hc{n}.in"]) and torch.equal(sub.join.put, Wt[f"{L}hc{n}.out"])
        assert torch.equal(sub.join.mix, Wt[f"{L}hc{n}.mix"]) and torch.equal(sub.conv[:, :W].t(), Wt[f"{L}canon{n}"]) and (sub.conv[:, W:] == 0).all()
    for i, (lay, spec) in enumerate(zip(m.layers, cfg["layers"])):
        L, s, f = f"l{i}.", spec["mixer"], spec["mlp"]
        p = L + "mix."
        check_sublayer(lay.mixer, L, 1)
        proj = xp @ lay.w_in.T + (lay.b_in if lay.b_in is not None else 0)
        if spec["type"] == "attention":
            gate = check_attention(lay.attention, s, p, proj, s["heads"] * lay.attention.dv).view(3, s["heads"], -1)
            assert same(gate[..., :s["vdim"]].reshape(3, -1), x @ Wt[p + "g"].T) and lay.attention.unit == s["dim"] and lay.delta is None
        else:
            s, r, H = s["left"], s["right"], s["left"]["heads"]
            gate = check_attention(lay.attention, s, p + "left.", proj[:, :lay.delta.col], up8(H))
            assert same(gate[:, :H], x @ Wt[p + "left.g"].T) and lay.attention.unit == 0
            per = H // s["kv_heads"]
            t = lay.attention.talk
            for h in range(H):
                for g in range(H):
                    assert t[g, h // per, h % per] == Wt[p + "left.talk"][h, g]
            assert (t[:, :, per:] == 0).all()
            d, p, (H, G, D, E) = lay.delta.weights, p + "right.", (r[k] for k in ("heads", "kv_heads", "dim", "vdim"))
            proj = proj[:, lay.delta.col:]
            q, k, v = proj[:, :d.col_b].split([G * d.dp, G * d.dp, H * d.vp], 1)
            cols = []
            for n, t, h, e, ep in (("q", q, G, D, d.dp), ("k", k, G, D, d.dp), ("v", v, H, E, d.vp)):
                t = t.reshape(3, h, ep)
                assert same(t[..., :e].reshape(3, -1), x @ Wt[p + n].T) and (t[..., e:] == 0).all()
                cols.append(torch.nn.functional.pad(Wt[f"{p}{n}.conv"].view(h, e, -1), (0, 0, 0, ep - e)).reshape(h * ep, -1))
            assert torch.equal(d.conv, torch.cat(cols).t())
            assert same(proj[:, d.col_b:d.col_b + H], x @ Wt[p + "b"].T) and same(proj[:, d.col_a:d.col_a + H], x @ Wt[p + "a"].T)
            g = proj[:, lay.delta.col_gate:].view(3, H, d.vp)
            assert same(g[..., :E].reshape(3, -1), x @ Wt[p + "g"].T) and (g[..., E:] == 0).all()
            assert torch.equal(d.a_log, Wt[p + "A_log"]) and torch.equal(d.dt_bias, Wt[p + "dt_bias"]) and torch.equal(d.norm[:E], Wt[p + "norm"])
            z = torch.randn(3, H, E)
            assert same((pad(z, d.vp).reshape(3, -1) @ lay.delta.o.T)[:, :W], z.reshape(3, -1) @ Wt[p + "o"].T)
            for nw, n in zip(lay.norms, ("left", "right")):
                assert torch.equal(nw.w[:W] * 2, Wt[f"{L}mix.{n}.out"])
        if f is None:
            assert lay.ff is None and lay.ffn is None
            continue
        check_sublayer(lay.ffn, L, 2)
        p = L + "mlp."
        if f["kind"] == "dense":
            assert same((xp @ lay.ff.up.T)[:, :f["ff"]], x @ Wt[p + "up"].T)
            z = torch.randn(3, f["ff"])
            assert same((pad(z, lay.ff.down.shape[1]) @ lay.ff.down.T)[:, :W], z @ Wt[p + "down"].T)
            a, b = ref.softplus(Wt[p + "act"].double()).tolist()
            assert abs(lay.ff.act[0] - a) < 1e-7 and abs(lay.ff.act[1] - 0.5 - b) < 1e-7
            continue
        assert same((xp @ lay.ff.router.T)[:, :f["router"]["experts"]], x @ Wt[p + "router"].T)
        for e in range(f["router"]["experts"]):
            ff = f["expert"]["ff"]
            gu = (xp @ lay.ff.up[e].T).view(3, -1, 2)[:, :ff]
            assert same(gu[..., 0], x @ Wt[f"{p}e{e}.gate"].T) and same(gu[..., 1], x @ Wt[f"{p}e{e}.up"].T)
            z = torch.randn(3, ff)
            assert same((pad(z, lay.ff.down.shape[2]) @ lay.ff.down[e].T)[:, :W], z @ Wt[f"{p}e{e}.down"].T)


def test_weight_errors():
    from inference_b200.contracts.errors import LoadError, Unsupported
    from inference_b200.models import ModelConfig
    from inference_b200.models.nafelix import NafelixGpu

    def load(w):
        return NafelixGpu(_cfg(), device=torch.device("cpu")).load_state_dict(w)
    good = ref.random_weights(ref.model_a())
    load(good)
    for name, t in (("head", None), ("l0.mix.left.talk", torch.zeros(6, 5)), ("l0.mix.right.q.conv", torch.zeros(48, 4)), ("l0.mlp.e3.up", None),
                    ("l0.hc1.mix", torch.zeros(3, 3)), ("l1.mix.q.b", None), ("l1.canon1", torch.zeros(144, 3)), ("l2.mlp.act", None),
                    ("l0.mix.right.out", None), ("l1.mix.g", torch.zeros(6, 144))):
        w = dict(good)
        if t is None:
            del w[name]
        else:
            w[name] = t
        with pytest.raises(LoadError):
            load(w)
    for edit in (lambda j: j.update(streams=17), lambda j: j["layers"][0]["mixer"]["right"].update(dim=513), lambda j: j["layers"][1]["mixer"].update(dim=1025)):
        j = ref.model_a()
        edit(j)
        with pytest.raises(Unsupported):
            NafelixGpu(ModelConfig.from_json(j), device=torch.device("cpu"))


def test_every_run_owns_pages_states_and_windows():
    from inference_b200.engine.kv_pool import LayeredKvPool, PagedSequence
    from inference_b200.models.registry import gpu_model

    m = gpu_model(_cfg(), device=torch.device("cpu"))
    pool = m.make_pool(6, 4, state_slots=3)
    shapes = [[tuple(t.shape) for t in kv] for kv in pool.data]
    canon = [(3, 3, 144)]
    first = [[(6, 3, 4, 40), (6, 1, 4, 72)], [(3, 6, 40, 32), (3, 2, 2 * 2 * 32 + 6 * 40)], canon, canon]
    looped = [[(6, 2, 4, 24), (6, 2, 4, 56)], canon, [(6, 1, 4, 24), (6, 1, 4, 40)], [(3, 3, 24, 64), (3, 3, 2 * 3 * 64 + 3 * 24)], canon, canon]
    assert shapes == first + looped * 3 + [[(6, 4, 4, 48), (6, 4, 4, 32)], canon, canon]
    assert m._places[:4] == [(0, 1, 2, 3), (4, 5, 5, 6), (6, 7, 8, 9), (10, 11, 11, 12)] and len(m._places) == 8 and m._places[-1] == (22, 23, 23, 24)
    per_token = 2 * (120 + 72 + 3 * (48 + 112 + 24 + 40) + 192 + 128)
    assert m.kv_block_bytes(4) == 4 * per_token == LayeredKvPool.block_bytes(m.kv_geometry(), 4, 2)
    # a copied state takes the windows along
    s = PagedSequence(pool)
    s.reserve(3)
    for kv in pool.data:
        for t in kv:
            if t.shape[0] == 3:
                t[s.state_slot] = 5.0
    other = (s.state_slot + 1) % 3
    pool.copy_state(s.state_slot, other)
    assert all((t[other] == 5).all() for kv in pool.data for t in kv if t.shape[0] == 3)
    s.release()
    assert pool.allocator.live_blocks() == pool.slots.live_blocks() == 0


def test_a_canon_of_one_tap_keeps_nothing():
    from inference_b200.models.registry import gpu_model

    m = gpu_model(_cfg("c"), device=torch.device("cpu"))
    pool = m.make_pool(2, 16, state_slots=1)
    assert pool.data[2][0].shape == (1, 0, 128)


def test_splits_follow_the_windows():
    from inference_b200.models.registry import gpu_model

    m = gpu_model(_cfg("d"), device=torch.device("cpu"))
    long, short = m.decode_splits(1, 100000), m.decode_splits(1, 1)
    assert long == m.decode_splits(1, 300) == (4, 2, 2) and short == (1, 1, 1)      # 263, 192 and 192 keys, 64 or 128 to a split at least
    assert m.decode_splits(500, 5000) == (1, 1, 1)
    plain = gpu_model(_cfg("d"), device=torch.device("cpu"), dtype=torch.float32)          # on the kernels with tiles of 64 keys
    assert plain.decode_splits(1, 100000) == (4, 2, 2) and plain.decode_splits(64, 100000) != m.decode_splits(64, 100000)


def test_exchange_behind_the_values():
    """Mixing the heads' weights and applying them equals applying every head's weights to all values and mixing the results."""
    g = torch.Generator().manual_seed(0)
    H, G, E = 6, 3, 4
    w, talk, v = (torch.rand(*s, generator=g, dtype=torch.float64) for s in ((H, 5, 9), (H, H), (9, G, E)))
    want = ref.apply_weights(ref.mix_heads(w, talk), v)
    a = torch.einsum("gts,sce->tgce", w, v)
    got = torch.stack([sum(talk[h, k] * a[:, k, h // (H // G)] for k in range(H)) for h in range(H)], 1)
    assert torch.allclose(got, want)


def _edit(path, fn):
    def go(cfg, w):
        for lay in cfg["layers"]:
            for m in [lay, lay["mixer"], {"mixer": lay["mixer"].get("left") or {}}]:
                d = m
                for p in path[:-1]:
                    d = d.get(p) or {}
                if path[-1] in d:
                    d[path[-1]] = fn(d[path[-1]])
        return cfg, w
    return go


def _change(suffix, fn):
    return lambda cfg, w: (cfg, {k: (fn(t) if k.endswith(suffix) else t) for k, t in w.items()})


def _patch(name, fn):
    """Replaces a function of the restatement."""
    return lambda cfg, w: (cfg, w, name, fn)


def _one_pass_less(cfg, w):
    cfg["loop"]["times"] -= 1
    return cfg, w


def _no_first_tokens(x, w):
    y = PLAIN_CONV(x, w)
    y[1:] += 0.5 * w[:, 0] * x[:1]             # what a window that is not cleared does
    return y


PLAIN_CONV, PLAIN_WRITE, PLAIN_ROUTE, PLAIN_EXPERT, PLAIN_TURN = (ref.causal_conv, ref.write_streams, ref.route, ref.clamped_expert,
                                                                  ref.rotate_halves)
MISTAKES = {
    "window one shorter": _edit(("mixer", "mask", "size"), lambda n: n - 1), "window one longer": _edit(("mixer", "mask", "size"), lambda n: n + 1),
    "scale": _edit(("mixer", "scale"), lambda s: s * 1.3), "base": _edit(("mixer", "rot", "base"), lambda b: b * 1.5),
    "one pass less": _one_pass_less, "no sink": _change("sink", lambda t: torch.full_like(t, -100.0)),
    "mixing transposed": _change("talk", lambda t: t.t().contiguous()), "streams transposed": _change("hc1.mix", lambda t: t.t().contiguous()),
    "streams of the feed-forward": _change("hc2.out", lambda t: t.roll(1)), "streams read": _change("hc2.in", lambda t: t.roll(1)),
    "no biases": _change("k.b", torch.zeros_like), "values' bias": _change("v.b", torch.zeros_like), "taps turned": _change("canon1", lambda t: t.flip(1)),
    "taps of the feed-forward": _change("canon2", lambda t: t.flip(1)), "taps of the delta rule": _change("k.conv", lambda t: t.flip(1)),
    "gate of the delta rule": _change("right.g", lambda t: t.roll(1, 0)), "gate per head": _change("left.g", lambda t: t.roll(1, 0)),
    "step size": _change("right.b", torch.zeros_like), "decay": _change("A_log", lambda t: t + 0.7), "decay's bias": _change("dt_bias", lambda t: t + 1),
    "halves swapped": _change("left.out", lambda t: t.roll(1)), "activation": _change("mlp.act", lambda t: t.flip(0)),
    "limit": _edit(("mlp", "expert", "limit"), lambda x: x * 1.5), "router": _change("router", lambda t: t.roll(1, 0)),
    "window kept from before": _patch("causal_conv", _no_first_tokens),
    "new streams used while joining": _patch("write_streams", lambda xs, mix, out, y: PLAIN_WRITE(PLAIN_WRITE(xs, mix, out, 0 * y), mix * 0 + torch.eye(len(mix)).to(mix), out, y * 0.9)),
    "scores as they are": _patch("route", lambda h, r, top: (PLAIN_ROUTE(h, r, top)[0], torch.softmax(h @ r.T, -1).gather(1, PLAIN_ROUTE(h, r, top)[0]))),
    "gate clamped from below": _patch("clamped_expert", lambda h, g, u, d, lim: (lambda a, b: (a * torch.sigmoid(1.702 * a) * (b + 1)) @ d.T)(
        torch.clamp(h @ g.T, -lim, lim), torch.clamp(h @ u.T, -lim, lim))),
    "neighbours rotated": _patch("rotate_halves", lambda x, pos, n, b: PLAIN_TURN(x.roll(1, -1), pos, n, b).roll(-1, -1)),
}


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_test_models_are_sensitive_to_mistakes(mistake, monkeypatch):
    """A mistake planted in the restatement moves the logits of the test models far beyond the tolerances of the GPU tests in 32-bit, and
    beyond those in bf16 for some positions."""
    tokens = torch.randint(0, 311, (60,), generator=torch.Generator().manual_seed(2)).tolist()
    cfg, w = ref.model_a(), ref.random_weights(ref.model_a(), seed=ord("a"))
    good = ref.forward(cfg, w, tokens)
    c, v, *patch = MISTAKES[mistake](copy.deepcopy(cfg), w)
    if patch:
        monkeypatch.setattr(ref, *patch)
    if mistake == "scores as they are":                  # with every expert chosen the scores sum to one: look at a layer that leaves some out
        c["layers"][0]["mlp"]["router"]["top"] = cfg["layers"][0]["mlp"]["router"]["top"] = 2
        monkeypatch.setattr(ref, "route", PLAIN_ROUTE)
        good = ref.forward(cfg, w, tokens)
        monkeypatch.setattr(ref, *patch)
    bad = ref.forward(c, v, tokens)
    err = (good - bad).square().mean(-1).sqrt() / good.square().mean(-1).sqrt()
    assert float(err.square().mean().sqrt()) > 0.02 and float(err.max()) > 0.05


def test_restatement_pieces():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)   # noqa: E731
    x, w = r(5, 2), r(2, 3)
    y = ref.causal_conv(x, w)
    assert torch.allclose(y[0], w[:, 2] * x[0]) and torch.allclose(y[4], w[:, 0] * x[2] + w[:, 1] * x[3] + w[:, 2] * x[4])
    # streams: from first index to second, all at once
    xs, mix, out, z = r(2, 3, 4), r(2, 2), r(2), r(3, 4)
    n = ref.write_streams(xs, mix, out, z)
    assert torch.allclose(n[1], mix[0, 1] * xs[0] + mix[1, 1] * xs[1] + out[1] * z)
    # rotation by halves: dimension 0 pairs with dims / 2, the rest stay
    e = torch.zeros(1, 1, 6, dtype=torch.float64)
    e[0, 0, 0], e[0, 0, 5] = 1.0, 7.0
    t = ref.rotate_halves(e, torch.tensor([2]), 4, 100.0)[0, 0]
    a = torch.tensor(2.0, dtype=torch.float64)
    assert torch.allclose(t, torch.stack([a.cos(), 0 * a, a.sin(), 0 * a, 0 * a, 7 + 0 * a]))
    # windows and sinks: a window of three sees itself and two before; a sink as large as the only score halves its weight
    q, k = r(1, 1, 4), r(8, 1, 4)
    seen = ref.attention_weights(q, k, torch.tensor([5]), 0.5, 3, None)[0, 0] > 0
    assert seen.tolist() == [False, False, False, True, True, True, False, False]
    one = ref.attention_weights(q, k, torch.tensor([5]), 0.5, 1, (q[:, 0] @ k[5, 0]) * 0.5)
    assert torch.allclose(one[0, 0, 5], torch.tensor(0.5, dtype=torch.float64))
    # a state that is read behind the write: with beta 1 and a unit key, reading with the key gives back the value
    key = torch.nn.functional.normalize(r(1, 1, 4), dim=-1)
    v = r(1, 1, 3)
    o, _ = ref.delta_rule(key, key, v, torch.ones(1, 1), torch.ones(1, 1, dtype=torch.float64), r(1, 4, 3))
    assert torch.allclose(o, v)
    pq = torch.tensor([0.3, -0.2], dtype=torch.float64)
    z = torch.tensor([2.0, -1.0, 0.0], dtype=torch.float64)
    sp = torch.log1p(torch.exp(pq))
    assert torch.allclose(ref.xielu(z, pq), torch.stack([sp[0] * 4 + 1, (0.5 + sp[1]) * (torch.exp(z[1]) - 1 + 1) - 0.5, 0 * sp[0]]))
    e, s = ref.route(r(3, 6), r(5, 6), 2)
    assert torch.allclose(s.sum(-1), torch.ones(3, dtype=torch.float64)) and e.shape == (3, 2)
    assert ref.margin(r(3, 6), r(4, 6), 4).isinf().all() and (ref.margin(r(3, 6), r(4, 6), 2) >= 0).all()
