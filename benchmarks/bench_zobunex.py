"""Zobunex beside the framework's sparse Llama-family decoder (Qwen2-MoE layers without a shared expert) at equal size.

Two parts, one JSON line per row:
  model   prefill and decode tokens/s of both decoders through the model runner (random weights). Both have the same width,
          layers, heads, vocabulary and expert parameters (an ungated Zobunex expert is 1.5 times as wide as a gated one);
          Zobunex attends in chunks as long as the context, so both read the same keys.
  kernel  every kernel of a Zobunex layer beside its counterpart: time, algorithmic bytes or FLOPs, and the fraction of the
          measured peak that is reached (MEASURED_PEAKS.json: copy bandwidth, bf16 GEMM).
CUDA events on the launching stream after warm-up; kernels with L2 flushed before every timed launch (a 512 MB write), models
with weights and caches larger than L2. Run as `python bench.py --design zobunex` or directly."""
import json
import statistics
import sys
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parent.parent
sys.path.insert(0, str(ROOT))

SIZES = {  # width, layers, heads, kv_heads, head dim, experts, top, gated ff, vocab
    "w2048_64x8": (2048, 12, 16, 4, 128, 64, 8, 1024, 32768),
    "w4096_8x2": (4096, 6, 32, 8, 128, 8, 2, 7168, 32768),
}
CHUNK = 2048


def peaks() -> tuple[float, float, str]:
    p = ROOT / "MEASURED_PEAKS.json"
    if p.is_file():
        d = json.loads(p.read_text())
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def zobunex_config(size, loop=None, dim=None):
    W, L, H, G, D, E, top, ff, V = SIZES[size]
    D = dim or D
    lay = {"type": "attention", "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "mask": {"size": CHUNK}, "scale": D ** -0.5,
                                          "rot": {"dims": D, "base": 10000.0}},
           "mlp": {"kind": "moe", "expert": {"ff": ff * 3 // 2}, "router": {"experts": E, "top": top}}}
    return {"architecture": "Zobunex", "width": W, "vocab": V, "norm": {"eps": 1e-5}, "logit_scale": 1.0, "loop": loop,
            "layers": [lay] * L}


def llama_config(size):
    W, L, H, G, D, E, top, ff, V = SIZES[size]
    return {"model_type": "qwen2_moe", "hidden_size": W, "intermediate_size": ff, "num_hidden_layers": L, "num_attention_heads": H,
            "num_key_value_heads": G, "head_dim": D, "vocab_size": V, "num_experts": E, "num_experts_per_tok": top,
            "moe_intermediate_size": ff, "shared_expert_intermediate_size": 0, "tie_word_embeddings": True}


def model_rows(size, which, cfg_json, emit):
    from inference_b200.engine.llm_engine import EngineConfig, LlmEngine
    from inference_b200.models import ModelConfig
    from inference_b200.models.registry import gpu_model

    cfg = ModelConfig.from_json(cfg_json)
    model = gpu_model(cfg, device=torch.device("cuda", 0)).init_random(seed=0)
    eng = LlmEngine(model, EngineConfig(max_batch=64, max_seq_len=1280))
    g = torch.Generator().manual_seed(1)
    prompts = [torch.randint(0, cfg.vocab_size, (1024,), generator=g).tolist() for _ in range(64)]

    def timed(fn, n=5):
        fn()
        fn()
        ms = []
        for _ in range(n):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            ms.append(a.elapsed_time(b))
        return statistics.median(ms)

    for B in (1, 8):
        def prefill():
            seqs = [eng.new_sequence() for _ in range(B)]
            eng.runner.prefill(seqs, prompts[:B])
            for s in seqs:
                s.release()
        ms = timed(prefill)
        emit({"part": "model", "size": size, "model": which, "what": f"prefill {B} x 1024", "ms": round(ms, 3),
              "tokens_per_s": round(B * 1024 / ms * 1e3), "launches": eng.runner.launches_last})
    for B in (1, 8, 64):
        seqs = [eng.new_sequence() for _ in range(B)]
        toks = []
        for i in range(0, B, 8):
            toks += eng.runner.prefill(seqs[i:i + 8], prompts[i:i + 8]).tolist()
        steps = 32

        def decode():
            eng.runner.decode_multi(seqs, toks, steps)
            for s in seqs:
                s.truncate(1024)
        ms = timed(decode) / steps
        emit({"part": "model", "size": size, "model": which, "what": f"decode batch {B}, context 1024", "ms": round(ms, 4),
              "tokens_per_s": round(B / ms * 1e3), "launches": eng.runner.launches_last // steps})
        for s in seqs:
            s.release()


def kernel_rows(size, emit):
    from inference_b200 import ops

    W, _, H, G, D, E, top, ff, V = SIZES[size]
    hbm, flops, _ = peaks()
    dev = "cuda"
    flush = torch.empty(512 << 20, dtype=torch.uint8, device=dev)
    gen = torch.Generator(device=dev).manual_seed(0)

    def rnd(*s, dtype=torch.bfloat16, std=1.0):
        return torch.empty(s, dtype=dtype, device=dev).normal_(0, std, generator=gen)

    def t(fn, n=15):
        for _ in range(3):
            fn()
        ev = []
        for _ in range(n):
            flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            ev.append(a.elapsed_time(b))
        return statistics.median(ev) * 1e-3

    def row(what, ours, like, our_work, like_work, kind):
        peak = hbm if kind == "bytes" else flops
        so, sl = t(ours), t(like)
        fo, fl = our_work / so / peak, like_work / sl / peak
        emit({"part": "kernel", "size": size, "what": what, "us": round(so * 1e6, 1), "like_us": round(sl * 1e6, 1), "bound": kind,
              "frac_of_peak": round(fo, 3), "like_frac_of_peak": round(fl, 3), "distance_ratio": round(fl / fo, 2)})

    # ---- residual + norm -------------------------------------------------------------------------------------------
    nw = ops.NormWeights(torch.ones(W, device=dev), torch.zeros(W, device=dev))
    w16 = torch.ones(W, dtype=torch.bfloat16, device=dev)
    for T in (64, 8192):
        x, y, h = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W)
        r16 = rnd(T, W)
        row(f"branch norm + residual + norm, T={T} (like: residual + RMS norm)",
            lambda: ops.stream_norm(x, W, 1e-5, branch=ops.Branch(y, nw), norm=nw, out=h),
            lambda: ops.rmsnorm(y, w16, 1e-5, residual=r16, out=h), T * W * 12, T * W * 8, "bytes")

    # ---- rotation and cache write -------------------------------------------------------------------------------------
    bs, T = 16, 8192
    cols = (H + 2 * G) * D
    qkv = rnd(T, cols)
    pos = (torch.arange(T, device=dev) % 2048).int()
    slots = torch.arange(T, device=dev)
    ang = torch.rand(2048, D // 2, device=dev)
    cos, sin = ang.cos().contiguous(), ang.sin().contiguous()
    kc, vc = torch.zeros(T // bs, G, bs, D, dtype=torch.bfloat16, device=dev), torch.zeros(T // bs, G, bs, D, dtype=torch.bfloat16, device=dev)
    moved = T * ((H + G) * D * 4 + 2 * G * D * 2 + G * D * 2)
    row("rotation + cache write, interleaved (like: half-split)",
        lambda: ops.rope_kv_write(qkv, pos, slots, cos, sin, kc, vc, H, G, D, interleaved=True, block_size=bs),
        lambda: ops.rope_kv_write(qkv, pos, slots, cos, sin, kc, vc, H, G, D, block_size=bs), moved, moved, "bytes")
    D9 = 96
    qkv9, kc9, vc9 = rnd(T, (H + 2 * G) * D9), kc[..., :D9].contiguous(), vc[..., :D9].contiguous()
    c9, s9 = cos[:, :D9 // 2].contiguous(), sin[:, :D9 // 2].contiguous()
    row("rotation + cache write, 96-wide heads (like: partial rotation of 128)",
        lambda: ops.rope_kv_write(qkv9, pos, slots, c9, s9, kc9, vc9, H, G, D9, interleaved=True, block_size=bs),
        lambda: ops.rope_kv_write(qkv, pos, slots, c9, s9, kc, vc, H, G, D, rot_dim=D9, interleaved=True, block_size=bs),
        moved * D9 // D, moved, "bytes")

    # ---- attention ------------------------------------------------------------------------------------------------------
    sink = torch.zeros(H, device=dev)
    tri = CHUNK * (CHUNK + 1) / 2
    pages = torch.randperm(T // bs, device=dev, generator=gen).int()
    cu1 = torch.tensor([0, T], dtype=torch.int32, device=dev)
    cu4 = torch.arange(0, T + 1, CHUNK, dtype=torch.int32, device=dev)
    lens1 = torch.tensor([T], dtype=torch.int32, device=dev)
    lens4 = torch.full((T // CHUNK,), CHUNK, dtype=torch.int32, device=dev)
    for d in (D, D9):
        qq, kk, vv = rnd(T, H, d), rnd(T, G, d), rnd(T, G, d)
        pk, pv = (kc, vc) if d == D else (kc9, vc9)
        q8, k8, v8 = rnd(T, H, D), rnd(T, G, D), rnd(T, G, D)
        work = 4.0 * H * d * tri * (T // CHUNK)
        like_work = 4.0 * H * D * tri * (T // CHUNK)
        row(f"chunked prefill attention, fresh, head width {d} (like: four causal sequences of one chunk, width {D})",
            lambda: ops.chunk_attention(qq, pk, pv, pages[None], lens1, cu_q=cu1, max_q_len=T, scale=d ** -0.5, chunk=CHUNK, sink=sink,
                                        fresh_kv=(kk, vv)),
            lambda: ops.varlen_causal_attention(q8, k8, v8, cu4, CHUNK, scale=D ** -0.5), work, like_work, "flops")
        row(f"chunked prefill attention, paged, head width {d} (like: four paged sequences of one chunk, width {D})",
            lambda: ops.chunk_attention(qq, pk, pv, pages[None], lens1, cu_q=cu1, max_q_len=T, scale=d ** -0.5, chunk=CHUNK, sink=sink),
            lambda: ops.paged_attention(q8, kc, vc, pages.view(T // CHUNK, -1), lens4, cu_q=cu4, max_q_len=CHUNK, scale=D ** -0.5),
            work, like_work, "flops")
    for B in (8, 64):
        ctx = 1024
        nb = B * ctx // bs
        table = torch.randperm(nb, device=dev, generator=gen).int().view(B, -1)
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        from inference_b200.models.llama import splits_for
        sp = splits_for(B, G, ctx)
        like_k, like_v = rnd(nb, G, bs, D), rnd(nb, G, bs, D)
        for d in (D, D9):
            k2, v2 = rnd(nb, G, bs, d), rnd(nb, G, bs, d)
            q2, q8 = rnd(B, H, d), rnd(B, H, D)
            row(f"decode attention, batch {B}, {ctx} visible keys, head width {d} (like: width {D})",
                lambda: ops.chunk_attention(q2, k2, v2, table, lens, cu_q=None, max_q_len=1, scale=d ** -0.5, chunk=CHUNK, sink=sink,
                                            decode=True, num_splits=sp),
                lambda: ops.paged_attention(q8, like_k, like_v, table, lens, cu_q=None, max_q_len=1, scale=D ** -0.5, decode=True,
                                            num_splits=sp),
                B * ctx * G * d * 4, B * ctx * G * D * 4, "bytes")

    # ---- experts --------------------------------------------------------------------------------------------------------
    from inference_b200.models import ModelConfig
    from inference_b200.models.llama import LlamaGpu, MoeWeights
    from inference_b200.models.zobunex import ZobunexGpu
    m = MoeWeights(rnd(E, W, std=0.02), rnd(E, 2 * ff, W, std=0.02), rnd(E, W, ff, std=0.02), None, None, None)
    like = LlamaGpu.__new__(LlamaGpu)
    like.cfg = ModelConfig.from_json(llama_config(size))
    fz = ff * 3 // 2
    up, down = rnd(E, fz, W, std=0.02), rnd(E, W, fz, std=0.02)
    table = torch.rand((V, E), generator=gen, device=dev).topk(top, 1).indices.int()[None].contiguous()
    for T in (1, 8, 64, 256, 1024, 8192):
        ids = torch.randint(0, V, (T,), generator=gen, device=dev)
        padded = T * top > ZobunexGpu.rows_per_expert_small * E
        plan = ops.table_routing(ids, table, E, padded=padded)[0]
        hx = rnd(T, W)
        h = rnd(plan.rows, W) if padded else hx
        used = int(table[0][ids].unique().numel())
        gpt = torch.softmax(hx.float() @ m.router.float().T, -1).topk(top, -1).indices
        like_used = int(gpt.unique().numel())
        big = T * top * W * fz * 4.0 / flops > used * W * fz * 4 / hbm
        wk = (T * top * W * fz * 4.0, T * top * W * ff * 6.0) if big else (used * W * fz * 4.0, like_used * W * ff * 6.0)
        row(f"experts, T={T} (like: router + sort + experts + combine)", lambda: ops.routed_ffn(h, up, down, plan, "relu2"),
            lambda: LlamaGpu._moe_ffn(like, hx, m), *wk, "flops" if big else "bytes")
        so = t(lambda: ops.table_routing(ids, table.expand(12, -1, -1).contiguous() if T == 1 else table, E, padded=padded))
        emit({"part": "kernel", "size": size, "what": f"routing plan, T={T}", "us": round(so * 1e6, 1)})


def main() -> int:
    if not torch.cuda.is_available():
        print(json.dumps({"error": "needs a CUDA device"}))
        return 1
    from inference_b200 import ops

    emit = lambda d: print(json.dumps(d), flush=True)   # noqa: E731
    hbm, fl, src = peaks()
    emit({"part": "peaks", "source": src, "hbm_gbs": hbm / 1e9, "bf16_tflops": fl / 1e12, "gpu": torch.cuda.get_device_name()})
    for size in SIZES:
        kernel_rows(size, emit)
        torch.cuda.empty_cache()
    for size in SIZES:
        model_rows(size, "zobunex", zobunex_config(size), emit)
        model_rows(size, "llama-moe", llama_config(size), emit)
        torch.cuda.empty_cache()
    model_rows("w2048_64x8", "zobunex, layers 2-9 twice", zobunex_config("w2048_64x8", {"start": 2, "stop": 10, "times": 2}), emit)
    ops.check_status()
    return 0


if __name__ == "__main__":
    sys.exit(main())
