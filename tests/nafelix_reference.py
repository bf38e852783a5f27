"""Plain, slow restatement of the Nafelix decoder in float64 on the CPU, one function per mechanism. It reads a config dict and a
name -> tensor dict and shares no code with the package; the GPU tests compare against it.

Also builds small random models for the tests. Their weights are drawn so that mistakes show: attention scores are peaked, sinks, gates
and clamps matter, head mixing and stream mixing are far from the identity, every convolution tap is of the same size, decays leave a
memory of some tens of tokens."""
from __future__ import annotations

import math

import torch

F = torch.float64


# ---- norms, stream ---------------------------------------------------------------------------------------------------
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def causal_conv(x, w):
    """x [T, C], w [C, taps]: y[t] = sum_j w[:, taps - 1 - j] x[t - j], zeros before the start."""
    taps = w.shape[1]
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(min(taps, t + 1)):
            y[t] += w[:, taps - 1 - j] * x[t - j]
    return y


def read_streams(xs, weights):
    """xs [S, T, W] -> sum_s weights[s] xs[s]."""
    return sum(weights[s] * xs[s] for s in range(xs.shape[0]))


def write_streams(xs, mix, out, y):
    """Every stream t becomes sum_s mix[s, t] xs[s] + out[t] y, from the old streams."""
    S = xs.shape[0]
    return torch.stack([sum(mix[s, t] * xs[s] for s in range(S)) + out[t] * y for t in range(S)])


# ---- attention -------------------------------------------------------------------------------------------------------
def rotate_halves(x, positions, dims, base):
    """x [T, heads, D]: (x_i, x_(i + dims/2)) turned by position * base^(-2i / dims) for i < dims / 2; the rest unchanged."""
    y = x.clone()
    n = dims // 2
    for i in range(n):
        a = positions.to(F) * float(base) ** (-2.0 * i / dims)
        c, s = a.cos()[:, None], a.sin()[:, None]
        u, v = x[:, :, i], x[:, :, i + n]
        y[:, :, i], y[:, :, i + n] = u * c - v * s, v * c + u * s
    return y


def attention_weights(q, k, q_pos, scale, window, sink):
    """q [T, H, D] at positions q_pos, k [S, G, D] at positions 0..S-1 -> weights [H, T, S]; sink [H] or None. window 0: none."""
    H, G = q.shape[1], k.shape[1]
    j = torch.arange(k.shape[0])[None]
    ok = j <= q_pos[:, None]
    if window:
        ok &= q_pos[:, None] - j < window
    out = torch.zeros(H, q.shape[0], k.shape[0], dtype=F)
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T * scale).masked_fill(~ok, -math.inf)
        top = s.max(-1).values
        if sink is not None:
            top = torch.maximum(top, sink[h].expand_as(top))
        e = torch.exp(s - top[:, None])
        den = e.sum(-1) + (torch.exp(sink[h] - top) if sink is not None else 0.0)
        out[h] = e / den[:, None]
    return out


def mix_heads(weights, talk):
    """weights [H, T, S] -> sum_g talk[h, g] weights[g]."""
    return torch.einsum("hg,gts->hts", talk, weights)


def apply_weights(weights, v):
    """weights [H, T, S], v [S, G, E]; head h reads value head h // (H / G) -> [T, H, E]."""
    H, G = weights.shape[0], v.shape[1]
    return torch.stack([weights[h] @ v[:, h // (H // G)] for h in range(H)], 1)


def talking_attention(h, W, p, m):
    """Windowed attention whose heads exchange their weights, one output gate per head; whole sequence."""
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q, k, v = ((h @ W[p + n].T).view(T, c, d) for n, c, d in (("q", H, D), ("k", G, D), ("v", G, E)))
    q, k = (rotate_halves(t, pos, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    w = mix_heads(attention_weights(q, k, pos, m["scale"], m["mask"]["size"], W[p + "sink"]), W[p + "talk"])
    a = apply_weights(w, v) * torch.sigmoid(h @ W[p + "g"].T)[..., None]
    return a.reshape(T, -1) @ W[p + "o"].T


def gated_attention(h, W, p, m, eps):
    """Windowed attention with biases, q and k of unit root mean square behind the rotation, a gate per output element; whole sequence."""
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q, k, v = ((h @ W[p + n].T + W[f"{p}{n}.b"]).view(T, c, d) for n, c, d in (("q", H, D), ("k", G, D), ("v", G, E)))
    q, k = (rms(rotate_halves(t, pos, m["rot"]["dims"], m["rot"]["base"]), eps) for t in (q, k))
    a = apply_weights(attention_weights(q, k, pos, m["scale"], m["mask"]["size"], W[p + "sink"]), v).reshape(T, -1)
    return (a * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---- delta rule ------------------------------------------------------------------------------------------------------
def silu(x):
    return x * torch.sigmoid(x)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def head_decay(x, a_log, dt_bias):
    """One per head: exp(-exp(A_log) softplus(x + dt_bias)), x [T, H]."""
    return torch.exp(-torch.exp(a_log) * torch.nn.functional.softplus(x + dt_bias))


def delta_rule(q, k, v, g, beta, state=None):
    """q / k [T, G, D], v [T, H, E], g and beta [T, H] -> (o [T, H, E], state [H, D, E])."""
    T, H, E = v.shape
    G, D = k.shape[1:]
    S = torch.zeros(H, D, E, dtype=F) if state is None else state.clone()
    o = torch.zeros(T, H, E, dtype=F)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // (H // G)], q[t, h // (H // G)]
            s = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - s.T @ kk)
            S[h] = s + torch.outer(kk, u)
            o[t, h] = S[h].T @ qq
    return o, S


def head_delta(h, W, p, m, eps):
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in "qkv")
    q, k = unit(q.view(T, G, D)) * D ** -0.5, unit(k.view(T, G, D))
    g = head_decay(h @ W[p + "a"].T, W[p + "A_log"], W[p + "dt_bias"])
    o, _ = delta_rule(q, k, v.view(T, H, E), g, torch.sigmoid(h @ W[p + "b"].T))
    o = rms(o, eps) * W[p + "norm"] * silu(h @ W[p + "g"].T).view(T, H, E)
    return o.reshape(T, -1) @ W[p + "o"].T


def parallel(h, W, p, m, eps):
    left = rms(talking_attention(h, W, p + "left.", m["left"]), eps) * W[p + "left.out"]
    right = rms(head_delta(h, W, p + "right.", m["right"], eps), eps) * W[p + "right.out"]
    return 0.5 * (left + right)


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def softplus(x):
    return torch.nn.functional.softplus(x)


def xielu(z, pq):
    a, b = softplus(pq[0]), 0.5 + softplus(pq[1])
    return torch.where(z > 0, a * z * z, b * (torch.expm1(z) - z)) + 0.5 * z


def clamped_expert(h, gate, up, down, limit):
    g, u = torch.clamp(h @ gate.T, max=limit), torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(h, router, top):
    """(experts, weights) [T, top]: the largest softmax scores, divided by their sum."""
    s, e = torch.sort(torch.softmax(h @ router.T, -1), dim=-1, descending=True, stable=True)
    s = s[:, :top]
    return e[:, :top], s / (s.sum(-1, keepdim=True) + 1e-20)


def margin(h, router, top):
    """Distance between the last chosen expert's logit and the first one left out [T] (inf when none is)."""
    z = torch.sort(h @ router.T, dim=-1, descending=True).values
    return z[:, top - 1] - z[:, top] if top < z.shape[1] else torch.full((h.shape[0],), math.inf, dtype=F)


def experts(h, W, p, f):
    e, s = route(h, W[p + "router"], f["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(e.shape[1]):
            q = f"{p}e{int(e[t, j])}."
            y[t] += s[t, j] * clamped_expert(h[t], W[q + "gate"], W[q + "up"], W[q + "down"], f["expert"]["limit"])
    return y


def feed_forward(h, W, p, f):
    if f["kind"] == "dense":
        return xielu(h @ W[p + "up"].T, W[p + "act"]) @ W[p + "down"].T
    return experts(h, W, p, f)


# ---- model -----------------------------------------------------------------------------------------------------------
def runs(cfg):
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return [*range(lp["start"]), *(list(range(lp["start"], lp["stop"])) * lp["times"]), *range(lp["stop"], n)]


def forward(cfg, weights, tokens, taps=None, margins=None):
    """Logits [T, vocab] of a whole sequence; `taps` collects the sum of the streams after every layer run, `margins` those of the routers."""
    W = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens)]
    xs = x[None].expand(cfg["streams"], -1, -1).clone()
    for i in runs(cfg):
        lay, L = cfg["layers"][i], f"l{i}."

        def sublayer(n, fn):
            h = rms(read_streams(xs, W[f"{L}hc{n}.in"]), eps) * W[f"{L}norm{n}"]
            return write_streams(xs, W[f"{L}hc{n}.mix"], W[f"{L}hc{n}.out"], fn(h + causal_conv(h, W[f"{L}canon{n}"])))
        mixer = {"parallel": parallel, "attention": gated_attention}[lay["type"]]
        xs = sublayer(1, lambda h: mixer(h, W, L + "mix.", lay["mixer"], eps))
        if lay["mlp"] is not None:
            def ff(h):
                if margins is not None and lay["mlp"]["kind"] == "moe":
                    margins.append(margin(h, W[L + "mlp.router"], lay["mlp"]["router"]["top"]))
                return feed_forward(h, W, L + "mlp.", lay["mlp"])
            xs = sublayer(2, ff)
        if taps is not None:
            taps.append(xs.sum(0))
    return (rms(xs.sum(0), eps) * W["final.norm"]) @ W["head"].T


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]


# ---- test models -----------------------------------------------------------------------------------------------------
def rot(dims, base):
    return {"dims": dims, "base": base}


def talk(heads, kv_heads, dim, vdim, window, rot_dims, base, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": rot(rot_dims, base),
            "scale": dim ** -0.5 if scale is None else scale}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def par(left, right):
    return "parallel", {"left": left, "right": right}


def attn(*args, **kw):
    return "attention", talk(*args, **kw)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(layers, width, vocab, streams, taps, loop=None, eps=1e-5):
    c = {"architecture": "Nafelix", "width": width, "vocab": vocab, "streams": streams, "canon": {"taps": taps}, "norm": {"eps": eps},
         "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def model_a():
    """Every layer different; groups of two and three heads, a layer without a feed-forward inside the loop."""
    return config([(par(talk(6, 3, 40, 24, 24, 24, 700.0), delta(6, 2, 24, 40, 3)), moe(4, 4, 24, 0.8)),
                   (attn(6, 2, 24, 56, 33, 8, 500.0), None),
                   (par(talk(4, 1, 24, 40, 17, 24, 90.0, scale=0.3), delta(3, 3, 40, 24, 4)), dense(120)),
                   (attn(4, 4, 48, 32, 70, 48, 2000.0), moe(5, 2, 56, 1.5))], 144, 311, 4, 4, loop=(1, 3, 3), eps=1e-3)


def model_b():
    """Nothing a multiple of eight, single heads, one expert for everyone, windows of one and two tokens, one stream, two taps."""
    return config([(par(talk(3, 3, 10, 7, 2, 6, 100.0), delta(1, 1, 5, 9, 2)), moe(3, 1, 13, 0.5)), (attn(1, 1, 14, 11, 1, 14, 30.0), dense(21)),
                   (par(talk(1, 1, 9, 5, 40, 2, 50.0), delta(2, 1, 33, 3, 1)), moe(1, 1, 7, 2.0))], 90, 77, 1, 2, eps=1e-2)


def model_c():
    """Widths beyond the tuned kernels: heads above 128, value heads that need several passes, seven streams, a canon of one tap."""
    return config([(par(talk(2, 2, 136, 136, 50, 100, 2000.0), delta(2, 1, 136, 72, 6)), dense(64)),
                   (attn(2, 1, 144, 132, 45, 64, 800.0), moe(9, 4, 16, 1.0)),
                   (par(talk(8, 4, 32, 64, 37, 16, 60.0), delta(4, 2, 16, 136, 4)), None)], 128, 150, 7, 1, loop=(2, 3, 2))


def model_d():
    """For long contexts: windows over page and tile borders, many heads on few keys, many experts."""
    return config([(par(talk(16, 2, 32, 64, 200, 32, 5e4), delta(8, 4, 32, 64, 4)), moe(40, 6, 16, 1.2)),
                   (attn(16, 1, 64, 96, 129, 16, 1e4), dense(136)),
                   (par(talk(12, 4, 64, 32, 129, 64, 1e4), delta(2, 2, 64, 64, 4)), moe(8, 8, 24, 0.7))], 256, 200, 2, 3)


MODELS = {"a": model_a, "b": model_b, "c": model_c, "d": model_d}


def random_weights(cfg, seed=0, peak=2.0):
    """bf16-representable weights; `peak` sets the spread of the attention scores."""
    g = torch.Generator().manual_seed(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * std + mean).to(torch.bfloat16)

    def lin(out, inp, std=1.0):
        return rnd(out, inp, std=std * inp ** -0.5)

    def qkv(p, m, bias):
        H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows, std in (("q", H * D, 1.0 if bias else peak / (m["scale"] * D ** 0.5)), ("k", G * D, 1.0), ("v", G * E, 1.0)):
            w[p + n] = lin(rows, W, std)
            if bias:
                w[f"{p}{n}.b"] = rnd(rows, std=0.5)
        w[p + "sink"] = rnd(H, std=1.0, mean=1.0)
        w[p + "g"] = lin(H * E if bias else H, W, 1.5)
        w[p + "o"] = lin(W, H * E)
    w = {"embed": rnd(V, W), "final.norm": rnd(W, std=0.3, mean=1.0), "head": lin(V, W, 2.0)}
    for i, lay in enumerate(cfg["layers"]):
        L, m, p, f = f"l{i}.", lay["mixer"], f"l{i}.mix.", lay["mlp"]
        for n in (1, 2) if f is not None else (1,):
            w[f"{L}norm{n}"] = rnd(W, std=0.3, mean=1.0)
            w[f"{L}canon{n}"] = rnd(W, cfg["canon"]["taps"], std=0.5)
            w[f"{L}hc{n}.in"], w[f"{L}hc{n}.out"] = rnd(S, std=0.5, mean=0.6), rnd(S, std=0.5, mean=0.6)
            w[f"{L}hc{n}.mix"] = ((torch.eye(S) * 0.7 + torch.randn(S, S, generator=g) * 0.4 * S ** -0.5)).to(torch.bfloat16)
        if lay["type"] == "attention":
            qkv(p, m, True)
        else:
            l, r = m["left"], m["right"]
            qkv(p + "left.", l, False)
            w[p + "left.talk"] = (torch.eye(l["heads"]) * 0.6 + torch.randn(l["heads"], l["heads"], generator=g) * 0.5).to(torch.bfloat16)
            H, G, D, E, q = r["heads"], r["kv_heads"], r["dim"], r["vdim"], p + "right."
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * E)):
                w[q + n], w[f"{q}{n}.conv"] = lin(rows, W, 2.0), rnd(rows, r["conv"], std=0.6)
            w[q + "b"], w[q + "a"], w[q + "g"] = lin(H, W, 1.5), lin(H, W), lin(H * E, W, 1.5)
            w[q + "A_log"], w[q + "dt_bias"] = rnd(H, std=0.5, mean=-1.0), rnd(H, std=0.5, mean=-1.5)
            w[q + "norm"], w[q + "o"] = rnd(E, std=0.3, mean=1.0), lin(W, H * E)
            w[p + "left.out"], w[p + "right.out"] = rnd(W, std=0.3, mean=1.0), rnd(W, std=0.3, mean=1.0)
        if f is None:
            continue
        p = L + "mlp."
        if f["kind"] == "dense":
            w[p + "up"], w[p + "down"], w[p + "act"] = lin(f["ff"], W), lin(W, f["ff"]), rnd(2, std=0.7)
            continue
        w[p + "router"] = lin(f["router"]["experts"], W, 2.0)
        for e in range(f["router"]["experts"]):
            ff = f["expert"]["ff"]
            w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff)
    return w
