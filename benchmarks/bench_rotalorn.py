"""Rotalorn beside the framework's Llama-family decoders at equal size.

Two parts, one JSON line per row:
  model   prefill and decode tokens/s through the model runner (random weights) at equal width, layers, heads, vocabulary and
          feed-forward parameters: routed layers beside Qwen2-MoE layers with a shared expert, dense layers beside dense Llama. Rotalorn
          stacks take the three mixers in turn; a stack of each mixer alone is timed as well. Windows are as long as the context, so that
          both models read the same keys.
  kernel  every kernel of a Rotalorn layer beside its counterpart: time, algorithmic bytes or FLOPs, and the fraction of the measured
          peak that is reached (MEASURED_PEAKS.json: copy bandwidth, bf16 GEMM). Windowed attention stands beside attention over as many
          visible keys: chunks of twice the window in prompts, a context of one window in decoding.
CUDA events on the launching stream after warm-up; kernels with L2 flushed before every timed launch (a 512 MB write), models
with weights and caches larger than L2. Run as `python bench.py --design rotalorn` or directly (an argument selects rows by name)."""
import dataclasses
import json
import statistics
import sys
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parent.parent
sys.path.insert(0, str(ROOT))

SIZES = {  # width, layers, heads, kv_heads, (experts, top, expert ff, shared ff) or None, dense ff, vocab
    "w2048_64x8": (2048, 12, 16, 4, (64, 8, 1024, 2048), 0, 32768),
    "w4096_dense": (4096, 6, 32, 8, None, 11264, 32768),
}
WINDOW = 2048


def rotalorn_config(size, pattern="LDA", window=WINDOW):
    """L latent attention, D differential attention, A grouped attention."""
    W, L, H, G, moe, ff, V = SIZES[size]
    mixers = {
        "L": ("latent_attention", {"heads": H, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": W // 2, "kv_rank": 512, "scale": 192 ** -0.5,
                                   "mask": {"size": window}, "rot": {"dims": 64, "base": 10000.0}}),
        "D": ("attention_2", {"heads": H, "kv_heads": G, "dim": 64, "vdim": 128, "scale": 0.125, "softcap": 30.0, "diff": 0.5,
                              "q_temp": {"coef": 0.1, "every": 4096}}),
        "A": ("attention", {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": window},
                            "rot": {"dims": 128, "base": 10000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}})}
    mlp = {"kind": "dense", "ff": ff}
    if moe:
        mlp = {"kind": "moe", "router": {"experts": moe[0], "top": moe[1]}, "expert": {"ff": moe[2]}, "shared": {"ff": moe[3]}}
    return {"architecture": "Rotalorn", "width": W, "vocab": V, "norm": {"eps": 1e-5},
            "embedding": {"bigram": {"buckets": 50021, "mul_prev": 31, "mul_cur": 17}},
            "layers": [{"type": mixers[k][0], "mixer": mixers[k][1], "mlp": mlp} for k in (pattern * L)[:L]]}


def llama_config(size):
    W, L, H, G, moe, ff, V = SIZES[size]
    c = {"hidden_size": W, "intermediate_size": ff or moe[2], "num_hidden_layers": L, "num_attention_heads": H, "num_key_value_heads": G,
         "head_dim": 128, "vocab_size": V, "tie_word_embeddings": True, "model_type": "llama"}
    if moe:
        c.update(model_type="qwen2_moe", num_experts=moe[0], num_experts_per_tok=moe[1], moe_intermediate_size=moe[2],
                 shared_expert_intermediate_size=moe[3])
    return c


def kernel_rows(size, emit, only=""):
    from benchmarks.bench_zobunex import peaks
    from inference_b200 import ops
    from inference_b200.models import ModelConfig
    from inference_b200.models.llama import LlamaGpu, MoeWeights, splits_for
    from inference_b200.models.rotalorn import RotalornGpu

    W, _, H, G, moe, ff, V = SIZES[size]
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
    peak = {"bytes": hbm, "flops": flops}

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

    bs, i32 = 16, lambda v: torch.tensor(v, dtype=torch.int32, device=dev)   # noqa: E731
    # ---- embedding and stream --------------------------------------------------------------------------------------------
    nw, w16 = ops.NormWeights(torch.ones(W, device=dev), torch.zeros(W, device=dev)), torch.ones(W, dtype=torch.bfloat16, device=dev)
    table, pairs = rnd(V, W), rnd(50022, W)
    for T in (64, 8192):
        x, y, h, r16 = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W), rnd(T, W)
        ids, pos, slots = torch.randint(0, V, (T,), generator=gen, device=dev), torch.arange(T, device=dev).int(), torch.arange(T, device=dev)
        pages, bt = torch.zeros((T // bs, bs), dtype=torch.int32, device=dev), torch.arange(T // bs, device=dev).int()[None].contiguous()
        row(f"embedding: token + pair rows into the fp32 stream, T={T} (like: embedding rows)",
            lambda: ops.stream_embed_pairs(ids, table, pairs, 31, 17, positions=pos, slots=slots, tokens=pages, block_table=bt, cu_q=None,
                                           num_seqs=1, max_q_len=T), T * W * 8, "bytes", lambda: ops.embedding(ids, table, out=h), T * W * 4)
        like = (lambda: ops.rmsnorm(y, w16, 1e-5, residual=r16, out=h), T * W * 8)
        row(f"stream: residual + layer norm, T={T} (like: residual + RMS norm)",
            lambda: ops.stream_norm(x, W, 1e-5, branch=ops.Branch(y, None), norm=nw, out=h), T * W * 12, "bytes", *like)
        if moe:
            E, top = moe[:2]
            ye = rnd(T * top, W)
            rr = ops.RoutedRows(ye, torch.randperm(T * top, device=dev, generator=gen).int().view(T, top), rnd(T, top, dtype=torch.float32))
            row(f"stream: the same + {top} weighted expert rows, T={T} (like: residual + RMS norm)",
                lambda: ops.stream_norm(x, W, 1e-5, branch=ops.Branch(y, None, extra=rr), norm=nw, out=h), T * W * (12 + 2 * top), "bytes", *like)
    # ---- preparation of queries, keys and values ------------------------------------------------------------------------------
    cos, sin = torch.ones(9000, 64, device=dev), torch.zeros(9000, 64, device=dev)
    c32, s32 = torch.ones(9000, 32, device=dev), torch.zeros(9000, 32, device=dev)
    for T in (64, 8192):
        pos, slots = (torch.arange(T, device=dev) % 1024).int(), torch.arange(T, device=dev)
        qkv, buf = rnd(T, (H + 2 * G) * 128), rnd(T, (H + 2 * G) * 128)
        kc, vc = rnd(T // bs, G, bs, 128), rnd(T // bs, G, bs, 128)
        qn, kn = torch.ones(H * 128, device=dev), torch.ones(G * 128, device=dev)
        like = (lambda: ops.rope_kv_write(qkv, pos, slots, cos, sin, kc, vc, H, G, 128, block_size=bs), T * ((H + G) * 512 + 3 * G * 256))
        row(f"whole-projection norms, rotation, raw values, cache write, T={T} (like: rotation + cache write)",
            lambda: ops.row_rope_kv_write(buf, pos, slots, kc, vc, H, G, 128, v_col=(H + G) * 128, rope=(cos, sin), q_norm=qn, k_norm=kn,
                                          norm_counts=(H * 128, G * 128), eps=1e-5, v_from_k=True), T * ((H + G) * 512 + 2 * G * 256), "bytes", *like)
        row(f"differential keys and values into the cache, T={T} (like: rotation + cache write)",
            lambda: ops.row_rope_kv_write(buf[:, H * 128:], pos, slots, kc, vc, 0, G, 128, v_col=G * 128), T * 2 * G * 512, "bytes", *like)
    # ---- latent attention -------------------------------------------------------------------------------------------------------
    base = rotalorn_config(size, "L")
    cfg = ModelConfig.from_json({**base, "layers": [{**base["layers"][0], "mlp": None}]})
    model = RotalornGpu(cfg, device=torch.device("cuda", 0)).init_random(seed=0)
    w = model.layers[0].latent
    T = 8192
    proj, pos, slots = rnd(T, model.layers[0].w_in.shape[0]), (torch.arange(T, device=dev) % 1024).int(), torch.arange(T, device=dev)
    cache, queries = rnd(T // bs, bs, w.width), rnd(T, H * (w.dn + w.rp))
    like = (lambda: ops.rope_kv_write(qkv, pos, slots, cos, sin, kc, vc, H, G, 128, block_size=bs), T * ((H + G) * 512 + 3 * G * 256))
    row("latent prep: both latents normed, key part rotated, cache write, T=8192 (like: rotation + cache write)",
        lambda: ops.latent_prep(proj, w, 1e-5, c32, s32, pos, slots, cache), T * (w.q_rank * 4 + 512 * 6 + 64 * 6), "bytes", *like)
    row("rotation of low-rank queries, T=8192 (like: rotation + cache write)", lambda: ops.rotate_queries(queries, w, c32, s32, pos),
        T * H * 64 * 4, "bytes", *like)
    a, kv, gate = rnd(T, H * w.vp), rnd(T, H * (w.dn + w.vp)), proj[:, w.col_gate:w.col_gate + H]
    q8, k8, v8 = rnd(T, H, 128), rnd(T, H, 128), rnd(T, H, 128)
    temp = torch.ones(9000, device=dev)

    def pairs_of(n, window):
        m = min(n, window)
        return m * (m + 1) / 2 + (n - m) * m
    for n, S, win in ((1024, 8, 0), (8192, 1, 0), (8192, 1, 1024), (8192, 1, 512)):
        cu = torch.arange(0, T + 1, n, dtype=torch.int32, device=dev)
        ww = dataclasses.replace(w, window=win)
        pr = S * pairs_of(n, win or n)
        bt, lens = torch.arange(T // bs, device=dev).int().view(S, -1).contiguous(), i32([n] * S)
        kp, vp = rnd(T // bs, G, bs, 128), rnd(T // bs, G, bs, 128)
        kf, vf = rnd(T, G, 128), rnd(T, G, 128)
        what, like = f"{S} x {n}", (lambda: ops.varlen_causal_attention(q8, k8, v8, cu, n, scale=0.1), 4.0 * H * 128 * pr, "flops")
        name = "causal"
        if win:
            what, name = f"{what}, window {win}", f"chunks of {2 * win}"
            like = (lambda: ops.chunk_attention(q8, kp, vp, bt, lens, cu_q=cu, max_q_len=n, scale=0.1, chunk=2 * win, fresh_kv=(kf, vf)),
                    4.0 * H * 128 * n * (2 * win + 1) / 2, "flops")
        row(f"latent prefill attention, {what}, q/k 128+64, v 128 (like: {name}, width 128)",
            lambda: ops.latent_prefill(queries, kv, proj[:, w.col_c + w.rk:w.col_gate], ww, a, cu_q=cu, max_q_len=n, gate=gate),
            2.0 * H * 320 * pr, "flops", *like)
        row(f"window prefill attention, {what}, width 128 (like: {name}, width 128)",
            lambda: ops.chunk_attention(q8, kp, vp, bt, lens, cu_q=cu, max_q_len=n, scale=0.1, window=win, fresh_kv=(kf, vf)),
            4.0 * H * 128 * pr, "flops", *like)
        if win:
            continue
        qd = rnd(T, H, 2, 64)
        for cap in (30.0, 0.0):
            d = ops.Differential(0.6, 0.5, 1e-5, 128, cap, temp)
            row(f"differential prefill attention, {what}, maps of 64, v 128, {'capped' if cap else 'uncapped'} (like: causal, width 128)",
                lambda: ops.chunk_attention(qd, kp, vp, bt, lens, cu_q=cu, max_q_len=n, scale=0.125, diff=d, fresh_kv=(kf, vf)),
                2.0 * H * 2 * (64 + 128) * pr, "flops", *like)
        d = ops.Differential(0.6, 0.5, 1e-5, 128, 30.0, temp)
        row(f"differential prefill attention from pages, {what}, capped (like: soft-capped paged kernel of the Llama family)",
            lambda: ops.chunk_attention(qd, kp, vp, bt, lens, cu_q=cu, max_q_len=n, scale=0.125, diff=d),
            2.0 * H * 2 * (64 + 128) * pr, "flops",
            lambda: ops.paged_attention(q8, kp, vp, bt, lens, cu_q=cu, max_q_len=n, scale=0.1, softcap=30.0), 4.0 * H * 128 * pr)
        wide = qd * 6.0
        row(f"differential prefill attention, {what}, scores beyond the cap (like: causal, width 128)",
            lambda: ops.chunk_attention(wide, kp, vp, bt, lens, cu_q=cu, max_q_len=n, scale=0.125, diff=d, fresh_kv=(kf, vf)),
            2.0 * H * 2 * (64 + 128) * pr, "flops", *like)
    for B, ctx, win in ((1, 1024, 0), (8, 1024, 0), (64, 1024, 0), (8, 8192, 0), (64, 8192, 1024), (64, 8192, 512)):
        nb = B * ctx // bs
        keys = win or ctx
        pool, tab = rnd(nb, bs, w.width), torch.randperm(nb, device=dev, generator=gen).int().view(B, -1)
        lens, seen = (torch.full((B,), n, dtype=torch.int32, device=dev) for n in (ctx, keys))
        q_abs, qq, qd = rnd(B, H, w.width), rnd(B, H, 128), rnd(B, H, 2, 64)
        lk, lv = rnd(nb, G, bs, 128), rnd(nb, G, bs, 128)
        spl, sw = splits_for(B, G, keys), splits_for(B, G, win + 63 if win else ctx)
        sp = model._latent_splits(dataclasses.replace(cfg.stack.layers[0].mixer, window=win), B, ctx)
        ww = dataclasses.replace(w, window=win)
        what = f"batch {B}, context {ctx}" + (f", window {win}" if win else "")
        like = (lambda: ops.paged_attention(qq, lk, lv, tab, seen, cu_q=None, max_q_len=1, scale=0.1, decode=True, num_splits=spl),
                B * keys * G * 512)
        name = f"(like: decode attention, {G} kv heads of 128, {keys} keys)"
        row(f"latent decode attention, {what} {name}",
            lambda: ops.latent_decode(q_abs, pool, tab, lens, ww, cu_q=None, max_q_len=1, num_splits=sp), B * keys * w.width * 2, "bytes", *like)
        row(f"window decode attention, {what} {name}",
            lambda: ops.chunk_attention(qq, lk, lv, tab, lens, cu_q=None, max_q_len=1, scale=0.1, window=win, decode=True, num_splits=sw),
            B * keys * G * 512, "bytes", *like)
        if not win:
            d = ops.Differential(0.6, 0.5, 1e-5, 128, 30.0, temp)
            row(f"differential decode attention, {what} {name}",
                lambda: ops.chunk_attention(qd, lk, lv, tab, lens, cu_q=None, max_q_len=1, scale=0.125, decode=True, num_splits=spl, diff=d),
                B * ctx * G * 512, "bytes", *like)
        if ctx > 1024:
            continue
        part = ops.latent_decode(q_abs, pool, tab, lens, w, cu_q=None, max_q_len=1, num_splits=sp)
        pj, oo, og, ps = rnd(B, H, w.dn + w.rp), rnd(B, H, w.vp), rnd(B, H), torch.zeros(B, dtype=torch.int32, device=dev)
        lw, lx = rnd(H * w.dn, w.rk), rnd(B, w.rk)
        like = (lambda: ops.gemm_bf16(lx, lw), H * w.dn * w.rk * 2)
        turn = ops.QueryRotation(c32, s32, ps, w.dn, w.rot, w.rp, w.rc)
        row(f"key projection + rotation of the queries, batch {B} (like: GEMM over as many weights)",
            lambda: ops.head_product(pj[..., :w.dn], w.uk_t, q_abs[..., :w.rk], rotate=turn), H * w.dn * w.rk * 2, "bytes", *like)
        row(f"split merge + value projection + gate, batch {B} (like: GEMM over as many weights)",
            lambda: ops.head_product(part, w.uv, oo, gate=og, sink=w.sink), H * w.vp * w.rk * 2 + part.o.nbytes, "bytes", *like)
        del pool, lk, lv
    # ---- feed-forward ---------------------------------------------------------------------------------------------------------------
    if not moe:
        for T in (8, 64, 8192):
            h, gu, out = rnd(T, W), rnd(2 * ff, W, std=0.02), torch.empty((T, ff + H * 128), dtype=torch.bfloat16, device=dev)
            work = (T * W * ff * 4.0, "flops") if T > 256 else (W * ff * 4.0, "bytes")
            row(f"gated projection into the joined activations, T={T} (like: into its own buffer)",
                lambda: ops.linear_gated(h, gu, "gelu", out=out[:, H * 128:]), *work, lambda: ops.linear_gated(h, gu, "silu"), work[0])
            wo, wd, wc = rnd(W, H * 128, std=0.02), rnd(W, ff, std=0.02), rnd(W, ff + H * 128, std=0.02)
            work = (T * W * (ff + H * 128) * 2.0, "flops") if T > 256 else (W * (ff + H * 128) * 2.0, "bytes")
            row(f"joined output projection, T={T} (like: two projections)", lambda: ops.gemm_bf16(out, wc), *work,
                lambda: (ops.gemm_bf16(out[:, :H * 128], wo), ops.gemm_bf16(out[:, H * 128:], wd)), work[0])
        return
    E, top, fe, fs = moe
    m = MoeWeights(rnd(E, W, std=0.02), rnd(E, 2 * fe, W, std=0.02), rnd(E, W, fe, std=0.02), None, None, None)
    like = LlamaGpu.__new__(LlamaGpu)
    like.cfg = ModelConfig.from_json(llama_config(size))
    router = torch.cat([m.router, rnd(8, W, std=0.02)])
    for T in (1, 8, 64, 256, 1024, 8192):
        h = rnd(T, W)
        spread = T * top > RotalornGpu.rows_per_expert_small * E

        def ours():
            logits = ops.gemm_bf16(h, router, out_dtype=torch.float32)
            plan, rows = ops.logits_routing(logits, E, top, rows=h if spread else None)
            return ops.routed_gated_ffn(rows if spread else h, m.gate_up, m.down, plan, "silu")
        used = int(torch.softmax(h.float() @ m.router.float().T, -1).topk(top, -1).indices.unique().numel())
        big = T * top * W * fe * 6.0 / flops > used * W * fe * 6 / hbm
        wk = T * top * W * fe * 6.0 if big else used * W * fe * 6.0
        row(f"router + experts, T={T} (like: router + sort + experts + combine)", ours, wk, "flops" if big else "bytes",
            lambda: LlamaGpu._moe_ffn(like, h, m), wk)
        logits = ops.gemm_bf16(h, router, out_dtype=torch.float32)
        row(f"routing from logits, T={T}", lambda: ops.logits_routing(logits, E, top, rows=h if spread else None),
            T * E * 4 + (T * top * W * 4 if spread else 0), "bytes")
        gu, out = rnd(T, 2 * fs), rnd(T, fs)
        row(f"gated activation + row gate, T={T} (like: gated activation)",
            lambda: ops.gated_act_mul(gu, "silu", out=out, paired=True, row_gate=logits[:, E]), T * fs * 6, "bytes",
            lambda: ops.gated_act_mul(gu, "silu", out=out, paired=True), T * fs * 6)


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
        model_rows(size, "rotalorn", rotalorn_config(size), emit)
        model_rows(size, "llama", llama_config(size), emit)
        torch.cuda.empty_cache()
    for pattern, what in (("L", "latent"), ("D", "differential"), ("A", "grouped")) if only in ("", "models") else ():
        model_rows("w4096_dense", f"rotalorn, all {what} attention", rotalorn_config("w4096_dense", pattern), emit)
        torch.cuda.empty_cache()
    ops.check_status()
    return 0


if __name__ == "__main__":
    sys.exit(main(sys.argv[1] if len(sys.argv) > 1 else ""))
