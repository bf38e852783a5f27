"""Plain, slow restatement of the Rotalorn decoder in float64 on the CPU, one function per mechanism. It reads a config dict and
a name -> tensor dict and shares no code with the package; the GPU tests compare against it.

Also builds small random models for the tests. Their weights are drawn so that mistakes show: attention scores are peaked, biases,
norm weights, gates and the second maps' share are not small, and the bigram rows are as large as the token rows."""
from __future__ import annotations

import math

import torch

F = torch.float64


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token of a sequence; the first token takes the extra row."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + t * mul_cur) % buckets for i, t in enumerate(tokens)]


def embedding(W, tokens, cfg):
    b = cfg["embedding"]["bigram"]
    return W["embed"][torch.tensor(tokens)] + W["bigram"][torch.tensor(bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]))]


def frequencies(rot):
    """Angle per position of every pair, with the long-context rescaling by wavelength when rot has `scaling`."""
    out, s = [], rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        if s is not None:
            wave = 2 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                mix = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1 - mix) * f / s["factor"] + mix * f
        out.append(f)
    return out


def rotate_halves(x, positions, rot):
    """x [T, heads, D]: dimension i < dims / 2 pairs with i + dims / 2; dimensions from dims on stay."""
    y, half = x.clone(), rot["dims"] // 2
    for i, f in enumerate(frequencies(rot)):
        a = positions.to(F) * f
        c, s = a.cos()[:, None], a.sin()[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i], y[:, :, i + half] = u * c - v * s, v * c + u * s
    return y


def visible(q_pos, keys, window):
    """[T, keys] mask: key j for the query at position i when 0 <= i - j, and i - j < window if there is one."""
    gap = q_pos[:, None] - torch.arange(keys)[None]
    return (gap >= 0) & ((gap < window) if window else True)


def softmax_attention(q, k, v, q_pos, scale, window=0, softcap=0.0):
    """q [T, H, D] at positions q_pos, k [S, H, D], v [S, H, E] at positions 0..S-1 -> [T, H, E]."""
    ok, out = visible(q_pos, k.shape[0], window), []
    for h in range(q.shape[1]):
        s = q[:, h] @ k[:, h].T * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        out.append(torch.softmax(s.masked_fill(~ok, -math.inf), -1) @ v[:, h])
    return torch.stack(out, 1)


def attention(h, W, p, m, eps):
    """Grouped heads; values are the keys as projected; norms over the whole projections, then rotation."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos, win = torch.arange(T), (m.get("mask") or {}).get("size", 0)
    q, k = h @ W[p + "q"].T + W[p + "q.b"], h @ W[p + "k"].T + W[p + "k.b"]
    v = k.view(T, G, D)
    q, k = rms(q, eps) * W[p + "q.norm"], rms(k, eps) * W[p + "k.norm"]
    q, k = (rotate_halves(t.view(T, -1, D), pos, m["rot"]) for t in (q, k))
    k, v = (t.repeat_interleave(H // G, 1) for t in (k, v))
    return softmax_attention(q, k, v, pos, m["scale"], win).reshape(T, -1) @ W[p + "o"].T


def latent_keys_values(c, k_rot, uk, uv, heads):
    """Latents [S, rank] and the shared rotated key part [S, rot] -> per-head keys [S, H, dim + rot], values [S, H, vdim]."""
    k = (c @ uk.T).view(c.shape[0], heads, -1)
    return torch.cat([k, k_rot[:, None].expand(-1, heads, -1)], -1), (c @ uv.T).view(c.shape[0], heads, -1)


def latent_attention(h, W, p, m, eps):
    T, H, D, R, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    pos, win = torch.arange(T), (m.get("mask") or {}).get("size", 0)
    low = rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (low @ W[p + "uq"].T).view(T, H, D + R)
    q = torch.cat([q[..., :D], rotate_halves(q[..., D:], pos, m["rot"])], -1)
    kv = h @ W[p + "dkv"].T
    c = rms(kv[:, :rank], eps) * W[p + "dkv.norm"]
    k, v = latent_keys_values(c, rotate_halves(kv[:, None, rank:], pos, m["rot"])[:, 0], W[p + "uk"], W[p + "uv"], H)
    a = softmax_attention(q, k, v, pos, m["scale"], win) * torch.sigmoid(h @ W[p + "g"].T)[..., None]
    return a.reshape(T, -1) @ W[p + "o"].T


def temperature(pos, coef, every):
    return 1 + coef * torch.log(torch.floor((pos.to(F) + 1) / every) + 1)


def second_map_share(W, p, diff):
    return torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum()) - torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum()) + diff


def differ(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1 - diff)


def differential_attention(h, W, p, m, eps):
    """Two softmax maps per head over the same values, the second subtracted."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(T)
    q, k = (h @ W[p + "q"].T).view(T, H, 2, D), (h @ W[p + "k"].T).view(T, G, 2, D).repeat_interleave(H // G, 1)
    v = (h @ W[p + "v"].T).view(T, G, -1).repeat_interleave(H // G, 1)
    q = q * temperature(pos, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None, None]
    a1, a2 = (softmax_attention(q[:, :, i], k[:, :, i], v, pos, m["scale"], 0, m["softcap"]) for i in (0, 1))
    return differ(a1, a2, second_map_share(W, p, m["diff"]), m["diff"], eps).reshape(T, -1) @ W[p + "o"].T


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def gated(h, W, p, act):
    return (act(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, router, top):
    """(experts [T, top], their softmax scores over all experts, as they are)."""
    s = torch.softmax(h @ router.T, -1)
    w, e = s.topk(top, -1)
    return e, w


def margin(h, router, top):
    """How far the last chosen expert's logit is above the first one left out (infinite when all are chosen)."""
    z = (h @ router.T).sort(-1, descending=True).values
    return z[:, top - 1] - z[:, top] if top < z.shape[1] else torch.full((len(h),), math.inf, dtype=F)


def mixture(h, W, p, f):
    """Routed experts plus the gated shared one."""
    e, w = route(h, W[p + "router"], f["router"]["top"])
    out = torch.sigmoid(h @ W[p + "shared.sg"].T) * gated(h, W, p + "shared.", silu)
    for t in range(h.shape[0]):
        for j in range(e.shape[1]):
            out[t] += w[t, j] * gated(h[t:t + 1], W, f"{p}e{int(e[t, j])}.", silu)[0]
    return out


MIXERS = {"attention": attention, "latent_attention": latent_attention, "attention_2": differential_attention}


def run(cfg, weights, tokens, margins=None):
    """Whole sequence at once: (logits [T, vocab], residual stream after every layer). `margins` collects the routers' margins."""
    W = {k: t.to(F) for k, t in weights.items()}
    eps, trail = cfg["norm"]["eps"], []
    norm = lambda x, n: layer_norm(x, W[n], W[n + ".b"], eps)   # noqa: E731
    x = embedding(W, tokens, cfg)
    for i, lay in enumerate(cfg["layers"]):
        L, f = f"l{i}.", lay["mlp"]
        h = norm(x, L + "norm1")
        if margins is not None and f is not None and f["kind"] == "moe":
            margins.append(margin(h, W[L + "mlp.router"], f["router"]["top"]))
        y = MIXERS[lay["type"]](h, W, L + "mix.", lay["mixer"], eps)
        if f is not None:
            y = y + (gated(h, W, L + "mlp.", gelu) if f["kind"] == "dense" else mixture(h, W, L + "mlp.", f))
        x = x + y
        trail.append(x)
    return norm(x, "final.norm") @ W["embed"].T, trail


def greedy(cfg, weights, prompt, steps):
    """Greedy continuation and, per step, the gap between the best and the second-best logit."""
    toks, gaps = list(prompt), []
    for _ in range(steps):
        top = run(cfg, weights, toks)[0][-1].topk(2)
        toks.append(int(top.indices[0]))
        gaps.append(float(top.values[0] - top.values[1]))
    return toks[len(prompt):], gaps


# ---- small random models --------------------------------------------------------------------------------------------
def attn(heads, kv_heads, dim, window, rot_dims, base, scaling=None, scale=None):
    rot = {"dims": rot_dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return ("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5 if scale is None else scale,
                          "mask": {"size": window}, "rot": rot})


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, base, scale=None):
    return ("latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                 "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "mask": {"size": window},
                                 "rot": {"dims": rot_dim, "base": base}})


def diffattn(heads, kv_heads, dim, vdim, softcap, coef, every, diff, scale=None):
    return ("attention_2", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": softcap, "diff": diff,
                            "q_temp": {"coef": coef, "every": every}, "scale": dim ** -0.5 if scale is None else scale})


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}


def config(layers, width, vocab, buckets, mul_prev, mul_cur, eps=1e-5):
    return {"architecture": "Rotalorn", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


def model_a():
    """Every layer different; partly rotated heads, groups of three, a layer without a feed-forward."""
    return config([(attn(6, 2, 40, 24, 24, 700.0, (8.0, 1.0, 4.0, 96)), moe(6, 3, 24, 40)), (diffattn(4, 2, 24, 40, 15.0, 0.3, 16, 0.35), dense(120)),
                   (latent(5, 24, 8, 40, 72, 48, 33, 900.0), moe(5, 2, 56, 24)), (diffattn(3, 3, 64, 128, 30.0, 0.7, 7, 0.8), None),
                   (attn(4, 4, 24, 17, 24, 50.0, scale=0.3), dense(72))], 144, 311, 97, 13, 29, eps=1e-3)


def model_b():
    """Nothing a multiple of eight, single heads, one expert for everyone, windows of one and two tokens."""
    return config([(latent(1, 18, 6, 14, 11, 20, 2, 100.0), moe(3, 1, 13, 5)), (attn(1, 1, 10, 1, 6, 30.0), dense(21)),
                   (diffattn(2, 1, 9, 7, 6.0, 1.5, 1, 0.1), moe(1, 1, 7, 9)), (diffattn(1, 1, 5, 12, 50.0, 0.0, 3, 0.0), dense(9))],
                  90, 77, 50, 7, 3, eps=1e-2)


def model_c():
    """Widths beyond the tuned kernels: heads above 128, maps above 64, values above 128, ranks above 512."""
    return config([(attn(2, 1, 136, 50, 100, 2000.0, (4.0, 1.0, 2.0, 64)), dense(64)), (diffattn(2, 1, 72, 56, 20.0, 0.4, 10, 0.5), moe(9, 4, 16, 24)),
                   (latent(2, 136, 72, 132, 40, 600, 40, 800.0), None), (diffattn(2, 2, 40, 136, 12.0, 0.2, 64, 0.6), dense(40))],
                  128, 150, 33, 5, 11)


def model_d():
    """For long contexts: wide windows over page and tile borders, many heads on few keys, many experts."""
    return config([(diffattn(16, 2, 32, 64, 25.0, 0.25, 100, 0.6), moe(40, 6, 16, 64)), (latent(20, 32, 32, 48, 96, 192, 200, 5e4), dense(136)),
                   (attn(16, 1, 64, 129, 64, 1e4, (8.0, 1.0, 4.0, 256)), moe(8, 8, 24, 16))], 256, 200, 500, 31, 17)


MODELS = {"a": model_a, "b": model_b, "c": model_c, "d": model_d}


def random_weights(cfg, seed=0, peak=2.0):
    """bf16-representable weights; `peak` sets the spread of the attention scores."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * std + mean).to(torch.bfloat16)

    def lin(out, inp, std=1.0):
        return rnd(out, inp, std=std * inp ** -0.5)

    def norm(n, size):
        w[n], w[n + ".b"] = rnd(size, std=0.3, mean=1.0), rnd(size, std=0.3)

    def ffn(p, ff, std=1.0):
        w[p + "gate"], w[p + "up"], w[p + "down"] = lin(ff, W, 1.5), lin(ff, W), lin(W, ff, std)
    w = {"embed": rnd(V, W), "bigram": rnd(cfg["embedding"]["bigram"]["buckets"] + 1, W)}
    norm("final.norm", W)
    for i, lay in enumerate(cfg["layers"]):
        L, m, p, f = f"l{i}.", lay["mixer"], f"l{i}.mix.", lay["mlp"]
        H, D = m["heads"], m["dim"]
        norm(L + "norm1", W)
        if lay["type"] == "attention":
            G = m["kv_heads"]
            for n, rows in (("q", H * D), ("k", G * D)):
                w[p + n], w[f"{p}{n}.b"], w[f"{p}{n}.norm"] = lin(rows, W), rnd(rows, std=0.5), rnd(rows, std=0.3, mean=1.0)
            w[p + "q.norm"] = (w[p + "q.norm"].float() * peak / (m["scale"] * D ** 0.5)).to(torch.bfloat16)
        elif lay["type"] == "latent_attention":
            R, E, rank, low = m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            w[p + "dq"], w[p + "dq.norm"] = lin(low, W), rnd(low, std=0.3, mean=1.0)
            w[p + "uq"] = lin(H * (D + R), low, peak / (m["scale"] * (D + R) ** 0.5))
            w[p + "dkv"], w[p + "dkv.norm"] = lin(rank + R, W), rnd(rank, std=0.3, mean=1.0)
            w[p + "uk"], w[p + "uv"], w[p + "g"] = lin(H * D, rank), lin(H * E, rank), lin(H, W, 1.5)
        else:
            G = m["kv_heads"]
            w[p + "q"] = lin(H * 2 * D, W, peak / (m["scale"] * D ** 0.5))
            w[p + "k"], w[p + "v"] = lin(G * 2 * D, W), lin(G * m["vdim"], W)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[p + n] = rnd(D, std=0.6 * D ** -0.25)
        w[p + "o"] = lin(W, H * m["vdim"])
        if f is None:
            continue
        if f["kind"] == "dense":
            ffn(L + "mlp.", f["ff"])
            continue
        E = f["router"]["experts"]
        w[L + "mlp.router"] = lin(E, W, 2.0)
        for e in range(E):
            ffn(f"{L}mlp.e{e}.", f["expert"]["ff"], 1.2)
        ffn(L + "mlp.shared.", f["shared"]["ff"])
        w[L + "mlp.shared.sg"] = lin(1, W, 1.5)
    return w
