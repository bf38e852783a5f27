"""Zobunex host side without a GPU: config reading, registry, weight checks and padding, cache geometry, replay protocol."""
import copy
import json

import pytest
import torch

import zobunex_reference as ref


def _cfg(name="a"):
    from inference_b200.models import ModelConfig

    return ModelConfig.from_json(ref.MODELS[name]())


def test_config_reads_every_size_and_constant():
    from inference_b200.models import Architecture

    c = _cfg()
    assert c.architecture is Architecture.ZOBUNEX and (c.hidden_size, c.vocab_size, c.rms_norm_eps) == (160, 321, 1e-3)
    m = c.stack.layers[2].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.chunk, m.rot_dims, m.rot_base, m.scale) == (2, 2, 128, 128, 50, 128, 3000.0, 0.07)
    assert c.stack.layers[1].mlp is None and c.stack.layers[3].mlp.ff == 72 and c.stack.logit_scale == 0.7
    for name in ref.MODELS:
        assert _cfg(name).stack.runs() == ref.schedule(ref.MODELS[name]())
    assert _cfg("c").groups == 20 and _cfg("c").stack.loop is None


@pytest.mark.parametrize("path,value", [(("width",), None), (("vocab",), 0), (("norm",), {}), (("layers", 0, "mixer", "heads"), 7),
                                        (("layers", 0, "mixer", "scale"), None), (("layers", 0, "mixer", "rot", "dims"), 25),
                                        (("loop", "stop"), 9), (("layers", 0, "mlp", "router", "top"), 0), (("layers",), [])])
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


def test_unknown_designs_layers_and_feed_forwards_are_refused():
    from inference_b200.contracts.errors import Unsupported
    from inference_b200.models import ModelConfig

    for edit in (lambda j: j.update(architecture="Other"), lambda j: j["layers"][0].update(type="scan"),
                 lambda j: j["layers"][0]["mlp"].update(kind="dense")):
        j = copy.deepcopy(ref.model_a())
        edit(j)
        with pytest.raises(Unsupported):
            ModelConfig.from_json(j)


def test_registry_and_providers(tmp_path):
    from inference_b200.contracts.core_llm import LoadSpec
    from inference_b200.contracts.errors import Unsupported
    from inference_b200.engine.provider import B200_LLAMA, CPU_LLAMA
    from inference_b200.models import ModelConfig
    from inference_b200.models.registry import gpu_model, gpu_supported
    from inference_b200.models.zobunex import ZobunexGpu

    cfg = _cfg()
    assert gpu_supported(cfg) and isinstance(gpu_model(cfg, device=torch.device("cpu")), ZobunexGpu)
    llama = ModelConfig.from_json({"hidden_size": 256, "intermediate_size": 256, "num_hidden_layers": 1, "vocab_size": 64,
                                   "num_attention_heads": 2, "head_dim": 128})
    with pytest.raises(Unsupported):
        gpu_model(llama, device=torch.device("cpu"), dtype=torch.float32)
    (tmp_path / "config.json").write_text(json.dumps(ref.model_a()))
    spec = LoadSpec.dense(str(tmp_path))
    assert B200_LLAMA.can_load(spec) and not CPU_LLAMA.can_load(spec)


@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_weights_land_padded_and_complete(name):
    from inference_b200.models.zobunex import ZobunexGpu

    cfg, w = ref.MODELS[name](), ref.random_weights(ref.MODELS[name]())
    m = ZobunexGpu(_cfg(name), device=torch.device("cpu"), dtype=torch.float32).load_state_dict(w)
    W = cfg["width"]
    assert m.hp % 8 == 0 and m.embed.shape == (cfg["vocab"], m.hp) and torch.equal(m.embed[:, :W], w["embed"].float())
    x = torch.randn(3, W)
    xp = torch.nn.functional.pad(x, (0, m.hp - W))
    for i, (lay, spec) in enumerate(zip(m.layers, cfg["layers"])):
        s = spec["mixer"]
        qkv = xp @ lay.qkv.T
        q = qkv[:, :s["heads"] * lay.dk].view(3, s["heads"], lay.dk)
        assert torch.allclose(q[..., :s["dim"]].reshape(3, -1), x @ w[f"l{i}.mix.q"].float().T, atol=1e-4)
        assert (q[..., s["dim"]:] == 0).all()
        a = torch.randn(3, s["heads"], s["vdim"])
        o = torch.nn.functional.pad(a, (0, lay.dv - s["vdim"])).reshape(3, -1) @ lay.o.T
        assert torch.allclose(o[:, :W], a.reshape(3, -1) @ w[f"l{i}.mix.o"].float().T, atol=1e-4) and (o[:, W:] == 0).all()
        if spec["mlp"]:
            key, k = lay.table
            assert torch.equal(m.tables[key][k], w[f"l{i}.mlp.table"])
    geo = m.kv_geometry()
    assert len(geo) == len(ref.schedule(cfg)) and all(g.k_dim % 8 == 0 and g.v_dim % 8 == 0 for g in geo)


def test_weight_errors():
    from inference_b200.contracts.errors import LoadError, Unsupported
    from inference_b200.models.zobunex import ZobunexGpu

    def load(w):
        return ZobunexGpu(_cfg(), device=torch.device("cpu")).load_state_dict(w)
    good = ref.random_weights(ref.model_a())
    load(good)
    for name, t in (("l0.mix.sink", None), ("loop.in", torch.zeros(3, 3)), ("l2.norm2b.b", None),
                    ("l0.mlp.table", good["l0.mlp.table"] + 5)):
        w = dict(good)
        if t is None:
            del w[name]
        else:
            w[name] = t
        with pytest.raises(LoadError):
            load(w)
    with pytest.raises(Unsupported):
        ZobunexGpu(_cfg(), device=torch.device("cpu"), dtype=torch.float16)


def test_layered_pool_shares_block_ids():
    from inference_b200.engine.kv_pool import KvGeometry, LayeredKvPool, PagedSequence

    geo = [KvGeometry(2, 16, 8), KvGeometry(1, 8, 24)]
    pool = LayeredKvPool(geo, 6, 4, device="cpu", dtype=torch.float32)
    assert pool.bytes == 6 * LayeredKvPool.block_bytes(geo, 4, 4)
    a, b = PagedSequence(pool), PagedSequence(pool)
    sa = a.reserve(6)
    b.reserve(9)
    assert len(set(a.blocks) & set(b.blocks)) == 0 and pool.allocator.free_blocks() == 1
    for kv in pool.data:
        for t in kv:
            t[a.blocks[1]] = 3.0
    c = PagedSequence.seeded(pool, list(a.blocks), 6)          # writing into the shared second page copies it everywhere
    c.reserve(1)
    assert c.blocks[0] == a.blocks[0] and c.blocks[1] != a.blocks[1]
    assert all(torch.equal(t[c.blocks[1]], t[a.blocks[1]]) for kv in pool.data for t in kv) and len(sa) == 6
    for s in (a, b, c):
        s.release()
    assert pool.allocator.live_blocks() == 0


class _Recorder:
    """A decode backend whose logits name the sequence and position they belong to."""
    vocab_size, max_context = 10, 8

    def __init__(self):
        self.live, self.made = set(), 0

    def new_sequence(self):
        self.made += 1
        s = {"id": self.made, "n": 0}
        self.live.add(self.made)
        return s

    def length(self, s):
        return s["n"]

    def release(self, s):
        self.live.discard(s["id"])

    def forward_at(self, seqs, toks, want):
        rows = []
        for s, t, w in zip(seqs, toks, want):
            rows += [[s["id"], s["n"] + k] + [0.0] * 8 for k in w]
            s["n"] += len(t)
        return torch.tensor(rows) if rows else None


def test_replay_protocol(tmp_path):
    from inference_b200.engine.trace_replay import replay

    b, done = _Recorder(), []
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": [1, 2, 3], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": [1], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": [4], "want": [0]}, {"id": "y", "tokens": [1, 1], "want": [1]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "x", "tokens": [5], "want": [0]}], "end": ["x", "y"]}]
    replay(b, [json.dumps(s) for s in lines] + [""], str(tmp_path), done.append)
    assert done == [0, 1, 2, 3] and not b.live and b.made == 3
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, 10)[:, :2].tolist()  # noqa: E731
    assert read(0) == [[1, 2], [1, 0]] and read(2) == [[1, 3], [2, 2]] and read(3) == [[3, 0]]
    assert not (tmp_path / "1.f32").exists()


@pytest.mark.parametrize("entry", [{"id": "x", "tokens": [10], "want": []}, {"id": "x", "tokens": [1], "want": [1]},
                                   {"id": "x", "tokens": [1] * 9, "want": []}])
def test_replay_refuses_bad_entries(tmp_path, entry):
    from inference_b200.engine.trace_replay import replay

    b = _Recorder()
    with pytest.raises(ValueError):
        replay(b, [json.dumps({"step": 0, "entries": [entry], "end": []})], str(tmp_path), lambda s: None)
    assert not b.live


def test_restatement_sees_chunk_edges_and_sinks():
    """The restatement itself: a key one position outside the chunk, or a sink left out, changes the result."""
    assert ref.visible(37, 37, 37) and not ref.visible(37, 36, 37) and ref.visible(36, 0, 37) and not ref.visible(3, 4, 0)
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(n, 2, 8, generator=g, dtype=torch.float64) for n in (1, 40, 40))
    at = torch.tensor([39])
    a = ref.attention(q, k, v, at, 0.5, 37, torch.zeros(2, dtype=torch.float64))
    manual = torch.stack([torch.softmax(torch.cat([q[0, h] @ k[37:, h].T * 0.5, torch.zeros(1, dtype=torch.float64)]), 0)[:-1] @ v[37:, h]
                          for h in range(2)])
    assert torch.allclose(a[0], manual)
    assert not torch.allclose(a, ref.attention(q, k, v, at, 0.5, 36, torch.zeros(2, dtype=torch.float64)), atol=1e-3)
    assert not torch.allclose(a, ref.attention(q, k, v, at, 0.5, 37, None), atol=1e-3)


def _drop(cfg, w, name, value):
    return cfg, {k: (torch.full_like(t, value) if k.endswith(name) else t) for k, t in w.items()}


def _chunks(cfg, w, by):
    for lay in cfg["layers"]:
        lay["mixer"]["mask"]["size"] += by
    return cfg, w


def _swap_loop(cfg, w):
    W = cfg["width"]
    return cfg, {**w, "loop.in": torch.cat([w["loop.in"][:, W:], w["loop.in"][:, :W]], 1)}


def _one_pass_less(cfg, w):
    cfg["loop"]["times"] -= 1
    return cfg, w


def _next_row(cfg, w):
    return cfg, {k: (t.roll(1, 0) if k.endswith("table") else t) for k, t in w.items()}


@pytest.mark.parametrize("mistake", [lambda c, w: _drop(c, w, ".sink", -60.0), lambda c, w: _chunks(c, w, 1),
                                     lambda c, w: _chunks(c, w, -1), lambda c, w: _drop(c, w, "norm1b.b", 0.0), _swap_loop,
                                     _one_pass_less, _next_row])
def test_test_models_are_sensitive_to_mistakes(mistake):
    """A mistake planted in the restatement moves the logits of the test models far beyond the tolerances of the GPU tests
    (3e-2 in bf16)."""
    tokens = torch.randint(0, 321, (139,), generator=torch.Generator().manual_seed(2)).tolist()
    cfg, w = ref.model_a(), ref.random_weights(ref.model_a(), seed=ord("a"))
    good = ref.run(cfg, w, tokens)[0]
    bad = ref.run(*mistake(copy.deepcopy(cfg), w), tokens)[0]
    assert float((good - bad).square().mean().sqrt() / good.square().mean().sqrt()) > 0.15
