"""Plain, slow restatement of the Gunedra decoder in float64 on the CPU, one function per mechanism. It reads a config dict
and a name -> tensor dict and shares no code with the package; the GPU tests compare against it.

Also builds small random models for the tests. Their weights are drawn so that mistakes show: attention scores are peaked,
sinks, gates and layer scales are not small, depth averages mix all earlier results, decays leave a memory of some tens of
tokens, and the delta rule's step sizes are spread over (0, 1)."""
from __future__ import annotations

import math

import torch

F = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x, w, groups, eps):
    """Every one of `groups` equal parts of the last axis by its own root mean square, then the weight."""
    parts = x.reshape(*x.shape[:-1], groups, -1)
    return rms(parts, eps).reshape(x.shape) * w


def rotate_pairs(x, positions, dims, base):
    """x [T, heads, D]: (x_2i, x_2i+1) turned by position * base^(-2i / dims) for 2i < dims; the rest unchanged."""
    y = x.clone()
    for i in range(dims // 2):
        a = positions.to(F) * float(base) ** (-2.0 * i / dims)
        c, s = a.cos()[:, None], a.sin()[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def sink_attention(q, k, v, q_pos, scale, sink):
    """q [T, H, D] at positions q_pos, k [S, H, D], v [S, H, E] at positions 0..S-1, causal -> [T, H, E]. sink [H] or None."""
    T, H, _ = q.shape
    ok = torch.arange(k.shape[0])[None] <= q_pos[:, None]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T * scale).masked_fill(~ok, -math.inf)
        top = s.max(-1).values
        if sink is not None:
            top = torch.maximum(top, sink[h].expand(T))
        e = torch.exp(s - top[:, None])
        den = e.sum(-1) + (torch.exp(sink[h] - top) if sink is not None else 0.0)
        out[:, h] = e @ v[:, h] / den[:, None]
    return out


def latent_keys_values(c, k_rot, uk, uv, heads):
    """Latents [S, rank] and the shared rotated key part [S, rot] -> per-head keys [S, H, dim + rot], values [S, H, vdim]."""
    k = (c @ uk.T).view(c.shape[0], heads, -1)
    return torch.cat([k, k_rot[:, None].expand(-1, heads, -1)], -1), (c @ uv.T).view(c.shape[0], heads, -1)


def latent_attention(h, W, p, m, eps):
    """Whole sequence; W maps names to tensors, `p` is the mixer's prefix."""
    T, H, D, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    pos = torch.arange(T)
    rot = lambda t: rotate_pairs(t, pos, m["rot"]["dims"], m["rot"]["base"])   # noqa: E731
    q = (h @ W[p + "q"].T).view(T, H, D + R)
    q = torch.cat([q[..., :D], rot(q[..., D:])], -1)
    low = h @ W[p + "dkv"].T
    c = rms(low[:, :m["kv_rank"]], eps) * W[p + "dkv.norm"]
    k, v = latent_keys_values(c, rot(low[:, None, m["kv_rank"]:])[:, 0], W[p + "uk"], W[p + "uv"], H)
    a = sink_attention(q, k, v, pos, m["scale"], W[p + "sink"])
    a = a * torch.sigmoid(h @ W[p + "g"].T)[..., None]
    return a.reshape(T, -1) @ W[p + "o"].T


def causal_conv_silu(x, w):
    """x [T, C], w [C, taps]: y[t] = silu(sum_j w[:, taps - 1 - j] x[t - j])."""
    taps = w.shape[1]
    xp = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F), x])
    y = sum(xp[i:i + x.shape[0]] * w[:, i] for i in range(taps))
    return y * torch.sigmoid(y)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta, state=None):
    """q / k [T, G, D], v [T, H, E], g [T, H, D] in (0, 1], beta [T, H] -> (o [T, H, E], state [H, D, E])."""
    T, H, E = v.shape
    G, D = k.shape[1:]
    S = torch.zeros(H, D, E, dtype=F) if state is None else state.clone()
    o = torch.zeros(T, H, E, dtype=F)
    for t in range(T):
        kk, qq = (a[t].repeat_interleave(H // G, 0) for a in (k, q))
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, kk))
        S = S + kk[:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hde,hd->he", S, qq)
    return o, S


def decay(x, a_log, dt_bias, heads):
    """exp(-exp(A_log) softplus(x + dt_bias)), x [T, heads * D] -> [T, heads, D]."""
    sp = torch.nn.functional.softplus(x + dt_bias).view(x.shape[0], heads, -1)
    return torch.exp(-torch.exp(a_log)[:, None] * sp)


def channel_delta(h, W, p, m, eps):
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv_silu(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q, k = unit(q.view(T, G, D)) * D ** -0.5, unit(k.view(T, G, D))
    beta = torch.sigmoid(h @ W[p + "b"].T)
    g = decay((h @ W[p + "a1"].T) @ W[p + "a2"].T, W[p + "A_log"], W[p + "dt_bias"], H)
    o, _ = delta_rule(q, k, v.view(T, H, E), g, beta)
    gate = torch.sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T).view(T, H, E)
    return (rms(o, eps) * W[p + "norm"] * gate).reshape(T, -1) @ W[p + "o"].T


def poly_norm(z, act, eps):
    return act[0] * rms(z, eps) + act[1] * rms(z ** 2, eps) + act[2] * rms(z ** 3, eps) + act[3]


def feed_forward(h, W, p, eps):
    return poly_norm(h @ W[p + "up"].T, W[p + "act"], eps) @ W[p + "down"].T


def depth_average(results, w):
    return sum(w[j] * x for j, x in enumerate(results))


MIXERS = {"latent_attention": latent_attention, "channel_delta": channel_delta}


def run(cfg, weights, tokens):
    """Whole sequence at once: (logits [T, vocab], residual stream after every layer)."""
    W = {k: t.to(F) for k, t in weights.items()}
    eps, groups, m = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["residual_mult"]
    norm = lambda x, n: grouped_norm(x, W[n], groups, eps)   # noqa: E731
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    results, trail = [x], []
    for i, lay in enumerate(cfg["layers"]):
        L = f"l{i}."
        y = MIXERS[lay["type"]](x, W, L + "mix.", lay["mixer"], eps)
        x = x + m * norm(y, L + "norm1") * W[L + "ls1"]
        if lay["mlp"] is not None:
            x = x + m * norm(feed_forward(x, W, L + "mlp.", eps), L + "norm2") * W[L + "ls2"]
        results.append(x)
        x = depth_average(results, W[L + "dwa"])
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
def latent(heads, dim, rot_dim, vdim, rank, base, scale=None):
    return ("latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
                                 "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": {"dims": rot_dim, "base": base}})


def delta(heads, kv_heads, dim, vdim, conv):
    return ("channel_delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv})


def config(layers, width, vocab, groups, eps=1e-5, residual_mult=0.5, embed_scale=1.0):
    return {"architecture": "Gunedra", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups},
            "residual_mult": residual_mult, "embedding": {"scale": embed_scale},
            "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (t, m), ff in layers]}


def model_a():
    """Every layer different; key heads shared by several value heads, a layer without a feed-forward, norm groups of 32."""
    return config([(latent(3, 40, 24, 56, 96, 500.0), 200), (delta(6, 3, 24, 40, 4), 56), (latent(5, 64, 16, 32, 128, 1e4, 0.2), None),
                   (delta(4, 4, 48, 24, 3), 72)], 160, 321, 5, eps=1e-3, residual_mult=0.7, embed_scale=1.7)


def model_b():
    """Nothing a multiple of eight, single heads, the shortest convolution with a window."""
    return config([(delta(2, 1, 10, 12, 2), 30), (latent(1, 18, 6, 14, 20, 100.0), 13), (delta(1, 1, 33, 7, 5), 21)], 90, 77, 3, eps=1e-2,
                  residual_mult=1.3)


def model_c():
    """Widths beyond the tuned kernels (attention heads above 128, rotated part above 64, rank above 512), no convolution window,
    one norm group."""
    return config([(latent(2, 136, 72, 132, 130, 2000.0), 64), (delta(2, 1, 140, 72, 1), None), (latent(3, 32, 8, 24, 600, 900.0), 24)],
                  256, 150, 1, embed_scale=0.5)


def model_d():
    """For long contexts: many heads on few latents, norm groups of whole 128-column chunks."""
    return config([(latent(20, 32, 32, 48, 192, 5e5), 300), (delta(4, 2, 64, 64, 4), 128), (latent(4, 128, 64, 128, 256, 1e4), 136)],
                  384, 200, 3, residual_mult=0.4, embed_scale=2.0)


def model_e():
    """Attention layers only: no recurrent state at all."""
    return config([(latent(2, 16, 8, 16, 64, 50.0), 40), (latent(4, 24, 16, 16, 40, 300.0), None)], 64, 90, 2)


def model_f():
    """Delta-rule layers only: no pages in use."""
    return config([(delta(2, 2, 16, 16, 4), 40), (delta(4, 1, 32, 8, 4), None)], 64, 90, 2)


MODELS = {"a": model_a, "b": model_b, "c": model_c, "d": model_d, "e": model_e, "f": model_f}


def random_weights(cfg, seed=0, peak=2.0):
    """bf16-representable weights; `peak` sets the spread of the attention scores."""
    g = torch.Generator().manual_seed(seed)
    W, V, s = cfg["width"], cfg["vocab"], cfg["embedding"]["scale"]

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * std + mean).to(torch.bfloat16)

    def lin(out, inp, std=1.0):
        return rnd(out, inp, std=std * inp ** -0.5)
    w = {"embed": rnd(V, W), "final.norm": rnd(W, std=0.3, mean=1.0)}
    for i, lay in enumerate(cfg["layers"]):
        L, m, p = f"l{i}.", lay["mixer"], f"l{i}.mix."
        for n in (1, 2) if lay["mlp"] else (1,):
            w[f"{L}norm{n}"], w[f"{L}ls{n}"] = rnd(W, std=0.3, mean=1.0), rnd(W, std=0.4, mean=0.8)
        w[L + "dwa"] = rnd(i + 2, std=0.3)
        w[L + "dwa"][-1] += 0.7
        H = m["heads"]
        if lay["type"] == "latent_attention":
            D, R, E, rank = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w[p + "q"] = lin(H * (D + R), W, peak / (m["scale"] * (D + R) ** 0.5 * max(s, 1.0)))
            w[p + "dkv"], w[p + "dkv.norm"] = lin(rank + R, W), rnd(rank, std=0.3, mean=1.0)
            w[p + "uk"], w[p + "uv"] = lin(H * D, rank), lin(H * E, rank)
            w[p + "sink"], w[p + "g"] = rnd(H, std=2.0), lin(H, W, 1.5)
        else:
            G, D, E = m["kv_heads"], m["dim"], m["vdim"]
            for n, c in (("q", G * D), ("k", G * D), ("v", H * E)):
                w[p + n], w[f"{p}{n}.conv"] = lin(c, W), rnd(c, m["conv"], std=m["conv"] ** -0.5)
            w[p + "b"], w[p + "A_log"], w[p + "norm"] = lin(H, W, 1.5), rnd(H, std=0.5, mean=-2.0), rnd(E, std=0.3, mean=1.0)
            ra, rg = max(3, D // 2 + 1), max(2, E // 3)
            w[p + "a1"], w[p + "a2"], w[p + "dt_bias"] = lin(ra, W), lin(H * D, ra), rnd(H * D, mean=-1.0)
            w[p + "g1"], w[p + "g2"] = lin(rg, W), lin(H * E, rg, 2.0)
        w[p + "o"] = lin(W, H * m["vdim"])
        if lay["mlp"]:
            ff = lay["mlp"]["ff"]
            w[L + "mlp.up"], w[L + "mlp.down"], w[L + "mlp.act"] = lin(ff, W), lin(W, ff), rnd(4, std=0.3, mean=0.5)
    return w
