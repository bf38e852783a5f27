"""Gunedra beside the framework's dense Llama-family decoder at equal size.

Two parts, one JSON line per row:
  model   prefill and decode tokens/s of both decoders through the model runner (random weights). Both have the same width,
          layers, heads, value width, vocabulary and feed-forward parameters (a Gunedra feed-forward is 1.5 times as wide as a
          gated one). Gunedra stacks mix latent attention and delta-rule layers; a stack of each kind alone is timed as well.
  kernel  every kernel of a Gunedra layer beside its counterpart: time, algorithmic bytes or FLOPs, and the fraction of the
          measured peak that is reached (MEASURED_PEAKS.json: copy bandwidth, bf16 GEMM; the recurrence is bound by the fp32
          FMA pipes in prompts: 148 SMs x 128 lanes x 2 at the measured clock limit). The recurrence has no counterpart: its
          rows stand beside the attention of the same step.
CUDA events on the launching stream after warm-up; kernels with L2 flushed before every timed launch (a 512 MB write), models
with weights and caches larger than L2. Run as `python bench.py --design gunedra` or directly."""
import json
import statistics
import sys
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parent.parent
sys.path.insert(0, str(ROOT))

SIZES = {  # width, layers, heads, dim, rot_dim, rank, vdim, gated ff, vocab
    "w2048": (2048, 12, 16, 128, 64, 512, 128, 5632, 32768),
    "w4096": (4096, 6, 32, 128, 64, 512, 128, 11264, 32768),
}
PATTERN = "LDLL"      # L latent attention, D delta rule


def gunedra_config(size, pattern=PATTERN):
    W, L, H, D, R, rank, E, ff, V = SIZES[size]
    mixers = {"L": ("latent_attention", {"heads": H, "dim": D, "rot_dim": R, "vdim": E, "kv_rank": rank, "scale": (D + R) ** -0.5,
                                         "rot": {"dims": R, "base": 10000.0}}),
              "D": ("channel_delta", {"heads": H, "kv_heads": H, "dim": D, "vdim": E, "conv": 4})}
    layers = [{"type": mixers[k][0], "mixer": mixers[k][1], "mlp": {"kind": "dense", "ff": ff * 3 // 2}}
              for k in (pattern * L)[:L]]
    return {"architecture": "Gunedra", "width": W, "vocab": V, "norm": {"eps": 1e-5, "groups": 2}, "embedding": {"scale": 16.0},
            "residual_mult": 0.3, "layers": layers}


def llama_config(size):
    W, L, H, D, R, rank, E, ff, V = SIZES[size]
    return {"model_type": "llama", "hidden_size": W, "intermediate_size": ff, "num_hidden_layers": L, "num_attention_heads": H,
            "num_key_value_heads": H // 4, "head_dim": 128, "vocab_size": V, "tie_word_embeddings": True}


def kernel_rows(size, emit, only=""):
    from benchmarks.bench_zobunex import peaks
    from inference_b200 import ops
    from inference_b200.models import ModelConfig
    from inference_b200.models.gunedra import GunedraGpu
    from inference_b200.models.llama import splits_for

    W, _, H, D, R, rank, E, ff, V = SIZES[size]
    hbm, flops, _ = peaks()
    fma = 148 * 128 * 2 * 1.965e9
    dev, F = "cuda", ff * 3 // 2
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
    peak = {"bytes": hbm, "flops": flops, "fma": fma}

    def row(what, ours, work, kind, like=None, like_work=None, like_kind=None):
        if only and only not in what:
            return
        so = t(ours)
        d = {"part": "kernel", "size": size, "what": what, "us": round(so * 1e6, 1), "bound": kind, "frac_of_peak": round(work / so / peak[kind], 3)}
        if like is not None:
            sl = t(like)
            fl = like_work / sl / peak[like_kind or kind]
            d.update(like_us=round(sl * 1e6, 1), like_frac_of_peak=round(fl, 3), distance_ratio=round(fl / (work / so / peak[kind]), 2))
        emit(d)

    # ---- stream ------------------------------------------------------------------------------------------------------
    nw, w16 = ops.NormWeights(torch.ones(W, device=dev)), torch.ones(W, dtype=torch.bfloat16, device=dev)
    for T in (64, 8192):
        x, y, h, r16 = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W), rnd(T, W)
        like = (lambda: ops.rmsnorm(y, w16, 1e-5, residual=r16, out=h), T * W * 8)
        row(f"stream: group norm of the branch + residual + copy, T={T} (like: residual + RMS norm)",
            lambda: ops.stream_norm(x, W, 1e-5, branch=ops.Branch(y, nw), out=h, center=False, groups=2), T * W * 12, "bytes", *like)
        n = 6
        hist, mix = rnd(n + 1, T, W, dtype=torch.float32), torch.full((n + 1,), 0.1, device=dev)
        row(f"stream: the same + depth average of {n + 1} results, T={T} (like: residual + RMS norm)",
            lambda: ops.stream_norm(x, W, 1e-5, branch=ops.Branch(y, nw), out=h, center=False, groups=2,
                                    average=ops.DepthAverage(hist, n, mix)), T * W * (16 + 4 * n), "bytes", *like)
        del hist
    # ---- feed-forward activation ---------------------------------------------------------------------------------------
    coef = torch.tensor([0.5, 0.3, 0.2, 0.1], device=dev)
    for T in (64, 8192):
        z, gu, o1, o2 = rnd(T, F), rnd(T, 2 * ff), rnd(T, F), rnd(T, ff)
        row(f"polynomial norm, T={T} (like: gated activation)", lambda: ops.poly_norm(z, coef, 1e-5, out=o1), T * F * 4, "bytes",
            lambda: ops.gated_act_mul(gu, out=o2), T * ff * 6)
    # ---- latent attention ------------------------------------------------------------------------------------------------
    cfg = ModelConfig.from_json({**gunedra_config(size), "layers": gunedra_config(size)["layers"][:2]})
    model = GunedraGpu(cfg, device=torch.device("cuda", 0)).init_random(seed=0)
    model.ensure_rope(9000)
    w, dl = model.layers[0].latent, model.layers[1]
    bs, G8 = 16, H // 4
    cos, sin = model._rope[model.layers[0].rope]
    cols = model.layers[0].w_in.shape[0]
    T = 8192
    proj, pos, slots = rnd(T, cols), (torch.arange(T, device=dev) % 1024).int(), torch.arange(T, device=dev)
    cache = rnd(T // bs, bs, w.width)
    kc, vc = rnd(T // bs, G8, bs, 128), rnd(T // bs, G8, bs, 128)
    qkv, c64, s64 = rnd(T, (H + 2 * G8) * 128), torch.ones(9000, 64, device=dev), torch.zeros(9000, 64, device=dev)
    moved = T * (H * R * 4 + rank * 6 + R * 4)
    row("latent prep (norm, rotation, cache write), T=8192 (like: rotation + cache write)",
        lambda: ops.latent_prep(proj, w, 1e-5, cos, sin, pos, slots, cache), moved, "bytes",
        lambda: ops.rope_kv_write(qkv, pos, slots, c64, s64, kc, vc, H, G8, 128, block_size=bs), T * ((H + G8) * 512 + 3 * G8 * 256))
    a = rnd(T, H * w.vp)
    kv = rnd(T, H * (w.dn + w.vp))
    gate = proj[:, w.col_gate:w.col_gate + H]
    q8, k8, v8 = rnd(T, H, 128), rnd(T, H, 128), rnd(T, H, 128)
    for n, S in ((1024, 8), (8192, 1)):
        cu = torch.arange(0, T + 1, n, dtype=torch.int32, device=dev)
        pairs = S * n * (n + 1) / 2
        row(f"latent prefill attention, {S} x {n}, q/k {D}+{R}, v {E} (like: causal, width 128)",
            lambda: ops.latent_prefill(proj[:, :w.col_c], kv, proj[:, w.col_c + w.rk:w.col_gate], w, a, cu_q=cu, max_q_len=n, gate=gate),
            2.0 * H * (D + R + E) * pairs, "flops", lambda: ops.varlen_causal_attention(q8, k8, v8, cu, n, scale=0.1), 4.0 * H * 128 * pairs)
    table = torch.randperm(T // bs, device=dev, generator=gen).int()[None].contiguous()
    ck = torch.tensor([0, T], dtype=torch.int32, device=dev)
    row("latent gather, 8192 rows", lambda: ops.latent_gather(cache, table, ck, T), T * w.width * 4, "bytes")
    row("latent expansion GEMM, 8192 rows", lambda: ops.gemm_bf16(cache.view(T, -1)[:, :w.rk], w.ukv), 2.0 * T * w.rk * H * (w.dn + w.vp), "flops")
    for B, ctx in ((1, 1024), (8, 1024), (64, 1024), (8, 8192), (64, 4096)):
        nb = B * ctx // bs
        pool, tab = rnd(nb, bs, w.width), torch.randperm(nb, device=dev, generator=gen).int().view(B, -1)
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        q_abs, qq = rnd(B, H, w.width), rnd(B, H, 128)
        lk, lv = rnd(nb, G8, bs, 128), rnd(nb, G8, bs, 128)
        sp, spl = model.decode_splits(B, ctx)[0], splits_for(B, G8, ctx)
        row(f"latent decode attention, batch {B}, context {ctx} (like: decode attention, {G8} kv heads of 128)",
            lambda: ops.latent_decode(q_abs, pool, tab, lens, w, cu_q=None, max_q_len=1, num_splits=sp), B * ctx * w.width * 2, "bytes",
            lambda: ops.paged_attention(qq, lk, lv, tab, lens, cu_q=None, max_q_len=1, scale=0.1, decode=True, num_splits=spl),
            B * ctx * G8 * 512)
        if ctx > 1024:
            continue
        part = ops.latent_decode(q_abs, pool, tab, lens, w, cu_q=None, max_q_len=1, num_splits=sp)
        pj, oo, og = rnd(B, H, w.dn + w.rp), rnd(B, H, w.vp), rnd(B, H)
        lw, lx = rnd(H * w.dn, w.rk), rnd(B, w.rk)
        like = (lambda: ops.gemm_bf16(lx, lw), H * w.dn * w.rk * 2)
        row(f"key projection of the queries, batch {B} (like: GEMM over as many weights)",
            lambda: ops.head_product(pj[..., :w.dn], w.uk_t, q_abs[..., :w.rk]), H * w.dn * w.rk * 2, "bytes", *like)
        row(f"split merge + value projection + gate, batch {B} (like: GEMM over as many weights)",
            lambda: ops.head_product(part, w.uv, oo, gate=og, sink=w.sink), H * w.vp * w.rk * 2 + part.o.nbytes, "bytes", *like)
        del pool, lk, lv
    # ---- delta rule --------------------------------------------------------------------------------------------------------
    d = dl.delta
    for B, n in ((1, 1024), (8, 1024), (1, 1), (8, 1), (64, 1)):
        T = B * n
        pj, dec, gt = rnd(T, dl.w_in.shape[0]), rnd(T, H * d.dp), rnd(T, H * d.vp)
        state, window = rnd(B, *d.state_shape(), dtype=torch.float32), rnd(B, *d.window_shape())
        slots, pos = torch.arange(B, device=dev).int(), (1 + torch.arange(T, device=dev) % n).int()
        cu = torch.arange(0, T + 1, n, dtype=torch.int32, device=dev)
        qq = rnd(T, H, 128)
        like = {}
        if n > 1:
            like = dict(like=lambda: ops.varlen_causal_attention(q8[:T], k8[:T], v8[:T], cu, n, scale=0.1),
                        like_work=4.0 * H * 128 * B * n * (n + 1) / 2, like_kind="flops")
            work, kind = 8.0 * T * H * d.dp * d.vp, "fma"
        else:
            nb = B * 1024 // bs
            lk, lv = rnd(nb, G8, bs, 128), rnd(nb, G8, bs, 128)
            tab, lens = torch.randperm(nb, device=dev, generator=gen).int().view(B, -1), torch.full((B,), 1024, dtype=torch.int32, device=dev)
            like = dict(like=lambda: ops.paged_attention(qq, lk, lv, tab, lens, cu_q=None, max_q_len=1, scale=0.1, decode=True,
                                                         num_splits=splits_for(B, G8, 1024)), like_work=B * 1024 * G8 * 512)
            work, kind = state.nbytes * 2, "bytes"
        row(f"delta rule with convolutions, norm and gate, {B} x {n} (like: attention of the step, context 1024)",
            lambda: ops.channel_delta(pj, dec, gt, d, 1e-5, state, window, slots, pos, cu_q=None, max_q_len=n), work, kind, **like)


def main(only: str = "") -> int:
    from benchmarks.bench_zobunex import model_rows, peaks

    if not torch.cuda.is_available():
        print(json.dumps({"error": "needs a CUDA device"}))
        return 1
    from inference_b200 import ops

    emit = lambda d: print(json.dumps(d), flush=True)   # noqa: E731
    hbm, fl, src = peaks()
    emit({"part": "peaks", "source": src, "hbm_gbs": hbm / 1e9, "bf16_tflops": fl / 1e12, "gpu": torch.cuda.get_device_name()})
    for size in SIZES:
        if only != "models":
            kernel_rows(size, emit, only)
        torch.cuda.empty_cache()
    for size in SIZES if only in ("", "models") else ():
        model_rows(size, "gunedra", gunedra_config(size), emit)
        model_rows(size, "llama", llama_config(size), emit)
        torch.cuda.empty_cache()
    for pattern, what in (("L", "latent attention"), ("D", "delta rule")) if only in ("", "models") else ():
        model_rows("w2048", f"gunedra, all {what}", gunedra_config("w2048", pattern), emit)
    ops.check_status()
    return 0


if __name__ == "__main__":
    sys.exit(main(sys.argv[1] if len(sys.argv) > 1 else ""))
