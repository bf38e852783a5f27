"""Nafelix beside the framework's closest decoders at equal size.

Two parts, one JSON line per row:
  model   prefill and decode tokens/s through the model runner (random weights) at equal width, layers, heads, vocabulary and feed-forward
          parameters: routed layers beside Rotalorn's (grouped attention in a window, routed experts) and Qwen2-MoE layers, dense ones beside
          Gunedra's delta-rule layers and dense Llama. Nafelix stacks alternate both mixers; a stack of each alone is timed as well. Windows
          are as long as the context, so that all read the same keys. Four streams, a convolution of four taps per sublayer.
  kernel  every kernel of a Nafelix layer beside its counterpart in the designs it shares the mechanism with: time, algorithmic bytes or
          FLOPs, and the fraction of the measured peak that is reached (MEASURED_PEAKS.json: copy bandwidth, bf16 GEMM; the delta rule in
          prompts against 128 fp32 lanes per SM at the maximum clock).
CUDA events on the launching stream after warm-up; kernels with L2 flushed before every timed launch (a 512 MB write), models with weights and
caches larger than L2. Run as `python bench.py --design nafelix` or directly (an argument selects rows by name)."""
import dataclasses
import json
import statistics
import sys
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parent.parent
sys.path.insert(0, str(ROOT))

SIZES = {  # width, layers, heads, kv_heads, (experts, top, expert ff) or None, gated dense ff, vocab
    "w2048_64x8": (2048, 12, 16, 4, (64, 8, 1024), 0, 32768),
    "w4096_dense": (4096, 6, 32, 8, None, 11264, 32768),
}
WINDOW, STREAMS, TAPS = 2048, 4, 4


def nafelix_config(size, pattern="PA"):
    """P parallel mixers, A gated attention. An ungated dense layer is 1.5 times as wide as a gated one."""
    W, L, H, G, moe, ff, V = SIZES[size]
    att = {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": WINDOW}, "rot": {"dims": 64, "base": 10000.0}}
    mixers = {"A": ("attention", att),
              "P": ("parallel", {"left": {**att, "vdim": 64}, "right": {"heads": H, "kv_heads": H // 2, "dim": 128, "vdim": 128, "conv": 4}})}
    mlp = {"kind": "dense", "ff": ff * 3 // 2}
    if moe:
        mlp = {"kind": "moe", "router": {"experts": moe[0], "top": moe[1]}, "expert": {"ff": moe[2], "limit": 7.0}}
    return {"architecture": "Nafelix", "width": W, "vocab": V, "norm": {"eps": 1e-5}, "streams": STREAMS, "canon": {"taps": TAPS},
            "layers": [{"type": mixers[k][0], "mixer": mixers[k][1], "mlp": mlp} for k in (pattern * L)[:L]]}


def rotalorn_config(size):
    W, L, H, G, moe, ff, V = SIZES[size]
    mix = {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": WINDOW}, "rot": {"dims": 64, "base": 10000.0}}
    mlp = {"kind": "moe", "router": {"experts": moe[0], "top": moe[1]}, "expert": {"ff": moe[2]}, "shared": {"ff": 64}}
    return {"architecture": "Rotalorn", "width": W, "vocab": V, "norm": {"eps": 1e-5},
            "embedding": {"bigram": {"buckets": 50021, "mul_prev": 31, "mul_cur": 17}}, "layers": [{"type": "attention", "mixer": mix, "mlp": mlp}] * L}


def gunedra_config(size):
    W, L, H, G, moe, ff, V = SIZES[size]
    mix = {"heads": H, "kv_heads": H // 2, "dim": 128, "vdim": 128, "conv": 4}
    return {"architecture": "Gunedra", "width": W, "vocab": V, "norm": {"eps": 1e-5, "groups": 2}, "embedding": {"scale": 4.0}, "residual_mult": 0.5,
            "layers": [{"type": "channel_delta", "mixer": mix, "mlp": {"kind": "dense", "ff": ff * 3 // 2}}] * L}


def llama_config(size):
    W, L, H, G, moe, ff, V = SIZES[size]
    c = {"hidden_size": W, "intermediate_size": ff or moe[2], "num_hidden_layers": L, "num_attention_heads": H, "num_key_value_heads": G,
         "head_dim": 128, "vocab_size": V, "tie_word_embeddings": True, "model_type": "llama"}
    if moe:
        c.update(model_type="qwen2_moe", num_experts=moe[0], num_experts_per_tok=moe[1], moe_intermediate_size=moe[2],
                 shared_expert_intermediate_size=0)
    return c


def kernel_rows(size, emit, only=""):
    from benchmarks.bench_zobunex import peaks
    from inference_b200 import ops
    from inference_b200.models import ModelConfig
    from inference_b200.models.llama import splits_for
    from inference_b200.models.nafelix import NafelixGpu

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
    peak = {"bytes": hbm, "flops": flops, "fma": 148 * 256 * 1.965e9}

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

    bs, i32, S = 16, lambda v: torch.tensor(v, dtype=torch.int32, device=dev), STREAMS   # noqa: E731
    # ---- streams and their convolution ---------------------------------------------------------------------------------------
    nw, nb_ = ops.NormWeights(torch.ones(W, device=dev)), ops.NormWeights(torch.ones(W, device=dev), torch.zeros(W, device=dev))
    join, read = ops.StreamMix(torch.eye(S, device=dev), torch.ones(S, device=dev)), torch.full((S,), 0.4, device=dev)
    for T in (8, 64, 8192):
        xs, x1, y, y2, h = rnd(T, S, W, dtype=torch.float32), rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W), rnd(T, W)
        slots, pos = torch.arange(T, device=dev).int(), torch.full((T,), 9, device=dev).int()
        conv = ops.ShortConv(rnd(TAPS, W, dtype=torch.float32), rnd(T if T <= 64 else 8, TAPS - 1, W))
        fused = dict(conv=conv, slots=slots, positions=pos) if T <= 64 else {}
        like = (lambda: ops.stream_norm(x1, W, 1e-5, branch=ops.Branch(y, None), norm=nb_, out=h), T * W * 12)
        base = T * W * (8 * S + 4) + (T * W * 4 * (TAPS - 1) if fused else 0)
        name = f"{S} streams: join, read, norm" + (", convolution" if fused else "")
        row(f"{name}, T={T} (like: residual + layer norm, one stream)",
            lambda: ops.hyper_step(xs, S, W, 1e-5, branch=ops.HyperBranch(y), join=join, x_out=xs, read=read, norm=nw, out=h, **fused), base, "bytes", *like)
        row(f"{name}, two normed branches, T={T} (like: residual + layer norm, one stream)",
            lambda: ops.hyper_step(xs, S, W, 1e-5, branch=ops.HyperBranch(y, nw, y2, nw), join=join, x_out=xs, read=read, norm=nw, out=h, **fused),
            base + T * W * 2, "bytes", *like)
        if moe:
            top = moe[1]
            ye = rnd(T * top, W)
            rr = ops.RoutedRows(ye, torch.randperm(T * top, device=dev, generator=gen).int().view(T, top), rnd(T, top, dtype=torch.float32))
            row(f"{name}, {top} weighted expert rows, T={T} (like: the same beside a dense row, one stream)",
                lambda: ops.hyper_step(xs, S, W, 1e-5, branch=ops.HyperBranch(rr), join=join, x_out=xs, read=read, norm=nw, out=h, **fused),
                base + T * W * 2 * (top - 1), "bytes",
                lambda: ops.stream_norm(x1, W, 1e-5, branch=ops.Branch(y, None, extra=rr), norm=nb_, out=h), T * W * (12 + 2 * top))
        if T > 64:
            cu = torch.arange(0, T + 1, 1024, dtype=torch.int32, device=dev)
            row(f"convolution of prompts, 8 x 1024 (like: residual + layer norm, one stream)",
                lambda: ops.short_conv(h, conv, slots[:8].contiguous(), pos, cu_q=cu, max_q_len=1024), T * W * 4, "bytes", *like)
    # ---- preparation, attention ------------------------------------------------------------------------------------------------
    cos, sin = torch.ones(9000, 32, device=dev), torch.zeros(9000, 32, device=dev)
    for T in (64, 8192):
        pos, slots = (torch.arange(T, device=dev) % 1024).int(), torch.arange(T, device=dev)
        a, b = rnd(T, (H + 2 * G) * 128), rnd(T, (H + 2 * G) * 128)
        kc, vc = rnd(T // bs, G, bs, 128), rnd(T // bs, G, bs, 128)
        v2 = rnd(T // bs, G // 2, bs, 128)
        qn, kn = torch.ones(H * 128, device=dev), torch.ones(G * 128, device=dev)
        like = (lambda: ops.row_rope_kv_write(b, pos, slots, kc, vc, H, G, 128, v_col=(H + G) * 128, rope=(cos, sin), q_norm=qn, k_norm=kn,
                                              norm_counts=(H * 128, G * 128), eps=1e-5, v_from_k=True), T * ((H + G) * 512 + 2 * G * 256))
        row(f"unit heads, rotation, cache write, T={T} (like: whole-projection norms, rotation, cache write)",
            lambda: ops.row_rope_kv_write(a, pos, slots, kc, vc, H, G, 128, v_col=(H + G) * 128, rope=(cos, sin), unit=128, eps=1e-5),
            T * ((H + G) * 512 + 3 * G * 256), "bytes", *like)
        row(f"rotation, cache write with narrow values, T={T} (like: whole-projection norms, rotation, cache write)",
            lambda: ops.row_rope_kv_write(a, pos, slots, kc, v2, H, G, 128, v_col=(H + G) * 128, rope=(cos, sin)),
            T * ((H + G) * 512 + G * 256 + G * 256), "bytes", *like)
    T, sink = 8192, torch.zeros(H, device=dev)
    q8, gate = rnd(T, H, 128), rnd(T, H * 128)
    talk = ops.head_mix_weights(torch.eye(H, device=dev), G)

    def pairs_of(n, window):
        m = min(n, window)
        return m * (m + 1) / 2 + (n - m) * m
    NV = G // 2                                           # value heads of 64, two to a tile
    base = nafelix_config(size, "P")
    model = NafelixGpu(ModelConfig.from_json({**base, "layers": [{**base["layers"][0], "mlp": None}]}), device=torch.device("cuda", 0)).init_random(seed=0)
    for n, B, win in ((1024, 8, 0), (8192, 1, 0), (8192, 1, 512)):
        cu = torch.arange(0, T + 1, n, dtype=torch.int32, device=dev)
        pr = B * pairs_of(n, win or n)
        bt, lens = torch.arange(T // bs, device=dev).int().view(B, -1).contiguous(), i32([n] * B)
        kp, vp, v2 = rnd(T // bs, G, bs, 128), rnd(T // bs, G, bs, 128), rnd(T // bs, NV, bs, 128)
        kf, vf, vf2 = rnd(T, G, 128), rnd(T, G, 128), rnd(T, NV, 128)
        what = f"{B} x {n}" + (f", window {win}" if win else "")
        kw = dict(cu_q=cu, max_q_len=n, scale=0.1, window=win)
        like = (lambda: ops.chunk_attention(q8, kp, vp, bt, lens, fresh_kv=(kf, vf), **kw), 4.0 * H * 128 * pr, "flops")
        row(f"prefill attention, sinks and element gates, {what} (like: the same without, width 128)",
            lambda: ops.chunk_attention(q8, kp, vp, bt, lens, fresh_kv=(kf, vf), sink=sink, gate=gate, **kw), 4.0 * H * 128 * pr, "flops", *like)
        row(f"prefill attention over all {G} value heads of 64, sinks, {what} (like: own values only, width 128)",
            lambda: ops.chunk_attention(q8, kp, v2, bt, lens, fresh_kv=(kf, vf2), sink=sink, all_values=True, **kw),
            2.0 * H * (128 + G * 64) * pr, "flops", *like)
        row(f"the same from pages, {what} (like: own values only, width 128)",
            lambda: ops.chunk_attention(q8, kp, v2, bt, lens, sink=sink, all_values=True, **kw),
            2.0 * H * (128 + G * 64) * pr, "flops", lambda: ops.chunk_attention(q8, kp, vp, bt, lens, **kw), 4.0 * H * 128 * pr)
    for T in (8, 64, 8192):
        a, g, maps, o = rnd(T, H, G, 64), rnd(T, H), rnd(T, H, 2, 128), rnd(T, H * 128)
        row(f"exchange of the heads' results and gates, T={T} (like: combination of differential maps)", lambda: ops.head_mix(a, talk, gate=g),
            T * H * (G + 1) * 128, "bytes", lambda: ops.diff_combine(maps, o, 0.5, 1e-5, 0.5), T * H * 768)
    for B, ctx, win in ((1, 1024, 0), (8, 1024, 0), (64, 1024, 0), (8, 8192, 0), (64, 8192, 512)):
        nb, keys = B * ctx // bs, win or ctx
        tab, lens = torch.randperm(nb, device=dev, generator=gen).int().view(B, -1), torch.full((B,), ctx, dtype=torch.int32, device=dev)
        qq, g = rnd(B, H, 128), rnd(B, H * 128)
        lk, lv, l2 = rnd(nb, G, bs, 128), rnd(nb, G, bs, 128), rnd(nb, NV, bs, 128)
        reach = win + 63 if win else ctx
        kw = dict(cu_q=None, max_q_len=1, scale=0.1, window=win, decode=True)
        what = f"batch {B}, context {ctx}" + (f", window {win}" if win else "")
        like = (lambda: ops.chunk_attention(qq, lk, lv, tab, lens, num_splits=splits_for(B, G, reach), **kw), B * keys * G * 512)
        row(f"decode attention, sinks and element gates, {what} (like: the same without)",
            lambda: ops.chunk_attention(qq, lk, lv, tab, lens, num_splits=splits_for(B, G, reach), sink=sink, gate=g, **kw),
            B * keys * G * 512, "bytes", *like)
        gh, ns = rnd(B, H), model.decode_splits(B, reach)[0]
        row(f"decode attention with exchanged weights, sinks and head gates, {what} (like: window attention, width 128)",
            lambda: ops.exchange_attention(qq, lk, l2, tab, lens, num_splits=ns, sink=sink, talk=talk, gate=gh, **kw), B * keys * G * 384, "bytes", *like)
    # ---- delta rule ----------------------------------------------------------------------------------------------------------------
    lay = model.layers[0]
    d = lay.delta.weights
    dc = dataclasses.replace(d, head_decay=False, dt_bias=torch.zeros(H * d.dp, device=dev))
    for B, n in ((1, 1024), (8, 1024), (1, 1), (8, 1), (64, 1)):
        T = B * n
        pj = rnd(T, lay.w_in.shape[0] - lay.delta.col)
        dec, gt = rnd(T, H * d.dp), rnd(T, H * d.vp)
        state, window = rnd(B, *d.state_shape(), dtype=torch.float32), rnd(B, *d.window_shape())
        slots, pos = torch.arange(B, device=dev).int(), (1 + torch.arange(T, device=dev) % n).int()
        work, kind = (8.0 * T * H * d.dp * d.vp, "fma") if n > 1 else (state.nbytes * 2, "bytes")
        row(f"delta rule, one decay per head, with convolutions, norm and gate, {B} x {n} (like: decays per key channel)",
            lambda: ops.head_delta(pj, gt, d, 1e-5, state, window, slots, pos, cu_q=None, max_q_len=n), work, kind,
            lambda: ops.channel_delta(pj, dec, gt, dc, 1e-5, state, window, slots, pos, cu_q=None, max_q_len=n), work)
    # ---- feed-forward --------------------------------------------------------------------------------------------------------------
    if not moe:
        F = ff * 3 // 2
        for T in (8, 64, 8192):
            h, up = rnd(T, W), rnd(F, W, std=0.02)
            work = (T * W * F * 2.0, "flops") if T > 256 else (W * F * 2.0, "bytes")
            row(f"projection with xIELU, T={T} (like: with squared relu)", lambda: ops.gemm_bf16(h, up, act="xielu", act_params=(0.7, 1.1)), *work,
                lambda: ops.gemm_bf16(h, up, act="relu2"), work[0])
        return
    E, top, fe = moe
    router, gu, down = rnd(E, W, std=0.02), rnd(E, 2 * fe, W, std=0.02), rnd(E, W, fe, std=0.02)
    for T in (1, 8, 64, 256, 1024, 8192):
        h = rnd(T, W)
        spread = T * top > NafelixGpu.rows_per_expert_small * E

        def ffn(act, **kw):
            logits = ops.gemm_bf16(h, router, out_dtype=torch.float32)
            plan, rows = ops.logits_routing(logits, E, top, rows=h if spread else None, **kw)
            return ops.routed_gated_ffn(rows if spread else h, gu, down, plan, act, 7.0)
        used = int(torch.softmax(h.float() @ router.float().T, -1).topk(top, -1).indices.unique().numel())
        big = T * top * W * fe * 6.0 / flops > used * W * fe * 6 / hbm
        wk = T * top * W * fe * 6.0 if big else used * W * fe * 6.0
        row(f"router + clamped experts, T={T} (like: gated experts, scores as they are)", lambda: ffn("clamped", renorm=True), wk,
            "flops" if big else "bytes", lambda: ffn("silu"), wk)


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
    for size, (_, _, _, _, moe, _, _) in SIZES.items() if only in ("", "models") else ():
        for which, cfg in (("nafelix", nafelix_config(size)), ("nafelix, all parallel", nafelix_config(size, "P")),
                           ("nafelix, all attention", nafelix_config(size, "A")),
                           ("rotalorn", rotalorn_config(size)) if moe else ("gunedra", gunedra_config(size)), ("llama", llama_config(size))):
            model_rows(size, which, cfg, emit)
            torch.cuda.empty_cache()
    ops.check_status()
    return 0


if __name__ == "__main__":
    sys.exit(main(sys.argv[1] if len(sys.argv) > 1 else ""))
