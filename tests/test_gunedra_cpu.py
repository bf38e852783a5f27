"""Gunedra host side without a GPU: config reading, registry, weight checks and padding, cache geometry, state slots, rollback and
forks of recurrent sequences, and whether the test models show mistakes."""
import copy
import json

import pytest
import torch

import gunedra_reference as ref


def _cfg(name="a"):
    from inference_b200.models import ModelConfig

    return ModelConfig.from_json(ref.MODELS[name]())


def test_config_reads_every_size_and_constant():
    from inference_b200.models import Architecture
    from inference_b200.models.config import ChannelDeltaSpec, DenseSpec, LatentAttentionSpec

    c = _cfg()
    assert c.architecture is Architecture.GUNEDRA and (c.hidden_size, c.vocab_size, c.rms_norm_eps) == (160, 321, 1e-3)
    s = c.stack
    assert (s.embed_scale, s.residual_mult, s.norm_groups, s.loop) == (1.7, 0.7, 5, None)
    assert s.layers[0].mixer == LatentAttentionSpec(3, 40, 24, 56, 96, 64 ** -0.5, 500.0) and s.layers[0].mlp == DenseSpec(200)
    assert s.layers[1].mixer == ChannelDeltaSpec(6, 3, 24, 40, 4)
    assert s.layers[2].mixer.scale == 0.2 and s.layers[2].mlp is None
    assert c.to_json() == ref.model_a() and c.groups == 5


@pytest.mark.parametrize("path,value", [(("width",), None), (("vocab",), 0), (("norm", "groups"), 7), (("norm", "eps"), None),
                                        (("residual_mult",), None), (("embedding",), None), (("layers", 0, "mixer", "scale"), None),
                                        (("layers", 0, "mixer", "rot_dim"), 23), (("layers", 0, "mixer", "rot", "dims"), 22),
                                        (("layers", 1, "mixer", "kv_heads"), 4), (("layers", 1, "mixer", "conv"), 0),
                                        (("layers", 1, "mlp", "ff"), None), (("layers",), [])])
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

    for edit in (lambda j: j["layers"][0].update(type="attention"), lambda j: j["layers"][1]["mlp"].update(kind="moe")):
        j = copy.deepcopy(ref.model_a())
        edit(j)
        with pytest.raises(Unsupported):
            ModelConfig.from_json(j)


def test_registry_and_providers(tmp_path):
    from inference_b200.contracts.core_llm import LoadSpec
    from inference_b200.engine.provider import B200_LLAMA, CPU_LLAMA
    from inference_b200.models.gunedra import GunedraGpu
    from inference_b200.models.registry import gpu_model, gpu_supported

    m = gpu_model(_cfg(), device=torch.device("cpu"))
    assert gpu_supported(_cfg()) and isinstance(m, GunedraGpu) and m.recurrent
    assert not gpu_model(_cfg("e"), device=torch.device("cpu")).recurrent
    (tmp_path / "config.json").write_text(json.dumps(ref.model_a()))
    spec = LoadSpec.dense(str(tmp_path))
    assert B200_LLAMA.can_load(spec) and not CPU_LLAMA.can_load(spec)


@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_weights_land_padded_and_complete(name):
    from inference_b200.models.gunedra import GunedraGpu

    cfg, w = ref.MODELS[name](), ref.random_weights(ref.MODELS[name]())
    m = GunedraGpu(_cfg(name), device=torch.device("cpu"), dtype=torch.float32).load_state_dict(w)
    W = cfg["width"]
    F = {k: t.float() for k, t in w.items()}
    x = torch.randn(3, W)
    xp = torch.nn.functional.pad(x, (0, m.hp - W))
    same = lambda a, b: torch.allclose(a, b, atol=1e-4)   # noqa: E731
    for i, (lay, spec) in enumerate(zip(m.layers, cfg["layers"])):
        s, p = spec["mixer"], f"l{i}.mix."
        H, proj = s["heads"], xp @ lay.w_in.T
        assert torch.allclose(lay.norm1.w[:W], F[f"l{i}.norm1"] * F[f"l{i}.ls1"] * cfg["residual_mult"])
        if spec["type"] == "latent_attention":
            z = lay.latent
            q = proj[:, :z.col_c].view(3, H, z.dn + z.rp)
            got = torch.cat([q[..., :s["dim"]], q[..., z.dn:z.dn + s["rot_dim"]]], -1)
            assert same(got.reshape(3, -1), x @ F[p + "q"].T) and (q[..., s["dim"]:z.dn] == 0).all()
            low = torch.cat([proj[:, z.col_c:z.col_c + z.rank], proj[:, z.col_c + z.rk:z.col_c + z.rk + z.rot]], -1)
            assert same(low, x @ F[p + "dkv"].T) and same(proj[:, z.col_gate:z.col_gate + H], x @ F[p + "g"].T)
            c = torch.randn(3, z.rank)
            cp = torch.nn.functional.pad(c, (0, z.rk - z.rank))
            assert same((cp @ z.uv.transpose(1, 2)).transpose(0, 1)[..., :s["vdim"]].reshape(3, -1), c @ F[p + "uv"].T)
            keys = torch.einsum("tr,hrd->thd", cp, z.uk_t)[..., :s["dim"]]
            assert same(keys.reshape(3, -1), c @ F[p + "uk"].T)
            assert torch.equal(z.ukv[:H * z.dn].view(H, z.dn, z.rk), z.uk_t.transpose(1, 2))
        else:
            z = lay.delta
            v = proj[:, 2 * z.kv_heads * z.dp:z.col_b].view(3, H, z.vp)
            assert same(v[..., :z.vdim].reshape(3, -1), x @ F[p + "v"].T) and same(proj[:, z.col_b:z.col_b + H], x @ F[p + "b"].T)
            for (col, up), n, d, dp in zip(lay.low, "ag", (z.dim, z.vdim), (z.dp, z.vp)):
                got = (proj[:, col:col + up.shape[1]] @ up.T).view(3, H, dp)
                assert same(got[..., :d].reshape(3, -1), x @ F[f"{p}{n}1"].T @ F[f"{p}{n}2"].T) and (got[..., d:] == 0).all()
            assert z.taps == s["conv"] and torch.equal(z.conv[:, :z.dim].t(), F[p + "q.conv"][:z.dim])
        a = torch.randn(3, H, s["vdim"])
        vp = lay.o.shape[1] // H
        o = torch.nn.functional.pad(a, (0, vp - s["vdim"])).reshape(3, -1) @ lay.o.T
        assert same(o[:, :W], a.reshape(3, -1) @ F[p + "o"].T) and (o[:, W:] == 0).all()


def test_weight_errors():
    from inference_b200.contracts.errors import LoadError, Unsupported
    from inference_b200.models import ModelConfig
    from inference_b200.models.gunedra import GunedraGpu

    def load(w):
        return GunedraGpu(_cfg(), device=torch.device("cpu")).load_state_dict(w)
    good = ref.random_weights(ref.model_a())
    load(good)
    for name, t in (("l0.mix.sink", None), ("l1.dwa", torch.zeros(4)), ("l1.mix.a2", torch.zeros(144, 5)), ("l0.ls2", None),
                    ("l3.mix.q.conv", torch.zeros(192, 4))):
        w = dict(good)
        if t is None:
            del w[name]
        else:
            w[name] = t
        with pytest.raises(LoadError):
            load(w)
    j = ref.model_a()
    j["layers"][1]["mixer"]["dim"] = 513
    with pytest.raises(Unsupported):
        GunedraGpu(ModelConfig.from_json(j), device=torch.device("cpu"))


def _pool(blocks=8, slots=3):
    from inference_b200.engine.kv_pool import LatentGeometry, LayeredKvPool, StateGeometry

    geo = [LatentGeometry(24), StateGeometry((2, 8, 4), (3, 10)), StateGeometry((1, 4, 4), (0, 6))]
    return LayeredKvPool(geo, blocks, 4, device="cpu", dtype=torch.bfloat16, state_slots=slots)


def test_pool_holds_pages_and_states():
    from inference_b200.engine.kv_pool import LayeredKvPool, PagedSequence
    from inference_b200.policy.paging import OutOfBlocks

    pool = _pool()
    assert [[tuple(t.shape) for t in kv] for kv in pool.data] == [[(8, 4, 24)], [(3, 2, 8, 4), (3, 3, 10)], [(3, 1, 4, 4), (3, 0, 6)]]
    assert pool.data[1][0].dtype == torch.float32 and pool.data[1][1].dtype == torch.bfloat16
    assert LayeredKvPool.block_bytes(pool.geometry, 4, 2) == 4 * 24 * 2
    seqs = [PagedSequence(pool) for _ in range(4)]
    for s in seqs[:3]:
        s.reserve(5)
    assert sorted(s.state_slot for s in seqs[:3]) == [0, 1, 2] and seqs[3].state_slot == -1
    with pytest.raises(OutOfBlocks):
        seqs[3].reserve(1)
    freed = seqs[1].state_slot
    seqs[1].release()
    seqs[3].reserve(1)
    assert seqs[3].state_slot == freed                         # slots and pages of a finished sequence are used again
    for s in seqs:
        s.release()
    assert pool.allocator.live_blocks() == 0 and pool.slots.live_blocks() == 0
    with pytest.raises(ValueError):
        LayeredKvPool(pool.geometry, 4, 4, device="cpu")


class _Runner:
    """Stands in for the model runner: the state of a sequence is the list of tokens it has seen, kept as a number per slot."""
    max_batch, max_seq_len = 8, 64

    def __init__(self, pool):
        self.pool, self.fed = pool, []
        self.model = type("M", (), {"cfg": type("C", (), {"vocab_size": 9})})

    def prefill(self, seqs, new_tokens, *, want=None, **kw):
        for s, toks in zip(seqs, new_tokens):
            start = s.length
            s.reserve(len(toks))
            st = self.pool.data[1][0][s.state_slot]
            if start == 0:
                st.zero_()
            for t in toks:
                st.copy_(st * 10 + t)
            s.fed(toks)
            self.fed.append(list(toks))
        return torch.zeros(sum(map(len, new_tokens)), 9) if want is None else None


    def decode(self, seqs, tokens, *, want_logits=False):
        self.prefill(seqs, [[t] for t in tokens])
        return torch.zeros(len(seqs), 9)


def _value(b, s):
    return float(b.runner.pool.data[1][0][s.state_slot].flatten()[0])


def test_rollback_restores_the_recurrent_state():
    from inference_b200.contracts.errors import Unsupported
    from inference_b200.engine.backend import GpuBackend

    b = GpuBackend(_Runner(_pool(slots=2)))
    s = b.new_sequence()
    b.forward([s], [[1, 2, 3]], all_positions=False)
    b.forward([s], [[4, 5, 6]], all_positions=True)            # a verify step: copies the state into the free slot first
    assert _value(b, s) == 123456 and s.checkpoint[0] == 3
    b.truncate(s, 4)
    assert (s.length, _value(b, s), s.tokens) == (4, 1234, [1, 2, 3, 4]) and b.runner.fed[-1] == [4]
    b.truncate(s, 2)                                           # in front of the checkpoint: rebuilt from the start
    assert (s.length, _value(b, s), b.runner.fed[-1]) == (2, 12, [1, 2])
    b.truncate(s, 0)
    b.forward([s], [[7]], all_positions=True)
    assert _value(b, s) == 7 and s.tokens == [7]
    s.fed(None)                                                # tokens chosen on the device
    s.reserve(2)
    with pytest.raises(Unsupported):
        b.truncate(s, 1)
    b.release(s)
    assert b.runner.pool.slots.live_blocks() == 0
    # without a free slot there is no checkpoint, and the state is rebuilt all the same
    t, u = b.new_sequence(), b.new_sequence()
    b.forward([t], [[1, 2]])
    b.forward([u], [[5]])
    b.forward([t], [[3, 4]], all_positions=True)
    assert t.checkpoint is None
    b.truncate(t, 3)
    assert _value(b, t) == 123 and _value(b, u) == 5


def test_forks_copy_the_state_of_a_sequence_as_it_stands():
    from inference_b200.engine.backend import GpuBackend

    b = GpuBackend(_Runner(_pool(slots=3)))
    s = b.new_sequence()
    b.forward([s], [[1, 2, 3, 4, 5]])
    f = b.fork(s, 5)
    assert b.length(f) == 5 and f.state_slot != s.state_slot and _value(b, f) == 12345 and f.blocks == s.blocks
    b.forward([f], [[6]])
    b.forward([s], [[7]])
    assert _value(b, f) == 123456 and _value(b, s) == 123457 and f.blocks[1] != s.blocks[1]    # the shared page was copied on write
    assert b.length(b.fork(s, 4)) == 0                          # an earlier state is gone
    g = b.fork(s, 6)
    assert b.length(g) == 6 and b.length(b.fork(s, 6)) == 0     # no slot left
    for x in (s, f, g):
        b.release(x)
    assert b.runner.pool.slots.live_blocks() == 0 and b.runner.pool.allocator.live_blocks() == 0


def _set(name, value):
    return lambda cfg, w: (cfg, {k: (torch.full_like(t, value) if k.endswith(name) else t) for k, t in w.items()})


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


def _top(fn):
    def go(cfg, w):
        fn(cfg)
        return cfg, w
    return go


def _roll(name, dim):
    return lambda cfg, w: (cfg, {k: (t.roll(1, dim) if k.endswith(name) else t) for k, t in w.items()})


@pytest.mark.parametrize("mistake", [_set(".sink", -60.0), _set("mix.g", 0.0), _set(".ls2", 1.0), _roll(".dwa", 0), _set("A_log", -9.0),
                                     _set("mix.b", 0.0), _roll(".conv", 1), _set("dt_bias", 0.0), _set("mix.g2", 0.0), _roll(".act", 0),
                                     _edit(("mixer", "rot", "base"), lambda b: b * 1.5), _edit(("mixer", "scale"), lambda s: s * 1.3),
                                     _top(lambda c: c.update(residual_mult=0.6)), _top(lambda c: c["embedding"].update(scale=1.2)),
                                     _top(lambda c: c["norm"].update(groups=1))])
def test_test_models_are_sensitive_to_mistakes(mistake):
    """A mistake planted in the restatement moves the logits of the test models far beyond the tolerances of the GPU tests."""
    tokens = torch.randint(0, 321, (60,), generator=torch.Generator().manual_seed(2)).tolist()
    cfg, w = ref.model_a(), ref.random_weights(ref.model_a(), seed=ord("a"))
    good = ref.run(cfg, w, tokens)[0]
    bad = ref.run(*mistake(copy.deepcopy(cfg), w), tokens)[0]
    assert float((good - bad).square().mean().sqrt() / good.square().mean().sqrt()) > 0.09


def test_restatement_pieces():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)   # noqa: E731
    # one step of the rule by hand, and the read-out sees the write
    k, q, v, dec, beta = r(1, 1, 3), r(1, 1, 3), r(1, 1, 2), torch.rand(1, 1, 3, generator=g, dtype=torch.float64), torch.tensor([[0.7]], dtype=torch.float64)
    S0 = r(1, 3, 2)
    o, S = ref.delta_rule(q, k, v, dec, beta, S0)
    D = S0[0] * dec[0, 0][:, None]
    want = D + torch.outer(k[0, 0], 0.7 * (v[0, 0] - D.T @ k[0, 0]))
    assert torch.allclose(S[0], want) and torch.allclose(o[0, 0], want.T @ q[0, 0])
    # convolution: the last column meets the current token
    y = ref.causal_conv_silu(torch.eye(3, dtype=torch.float64)[:, :1], torch.tensor([[2.0, 3.0]], dtype=torch.float64))
    z = torch.tensor([3.0, 2.0, 0.0], dtype=torch.float64)
    assert torch.allclose(y[:, 0], z * torch.sigmoid(z))
    x = r(2, 6)
    n = ref.grouped_norm(x, torch.ones(6, dtype=torch.float64), 2, 0.0)
    assert torch.allclose(n[:, :3].square().mean(-1), torch.ones(2, dtype=torch.float64))
    a = ref.sink_attention(r(1, 1, 4), r(5, 1, 4), torch.ones(5, 1, 1, dtype=torch.float64), torch.tensor([4]), 0.5, torch.zeros(1, dtype=torch.float64))
    assert 0 < float(a) < 1
