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
