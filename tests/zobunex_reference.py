"""Plain, slow restatement of the Zobunex decoder in float64 on the CPU, one function per mechanism. It reads a config
dict and a name -> tensor dict and shares no code with the package; the GPU tests compare against it.

Also builds small random models for the tests. Their weights are drawn so that mistakes show: query / key projections are
large (attention weights are peaked, so one key more or less changes the result), sinks and norm biases are not small, and
every table row names different experts."""
from __future__ import annotations

import math

import torch

F = torch.float64


def layer_norm(x, w, b, eps):
    mu = x.mean(-1, keepdim=True)
    d = x - mu
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotate_pairs(x, positions, dims, base):
    """x [T, heads, D]: (x_2i, x_2i+1) turned by position * base^(-2i / dims) for 2i < dims; the rest unchanged."""
    y = x.clone()
    for i in range(dims // 2):
        a = positions.to(F) * float(base) ** (-2.0 * i / dims)
        c, s = a.cos()[:, None], a.sin()[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def visible(i, j, chunk):
    """Whether the query at position i sees the key at position j."""
    return j <= i and (not chunk or i // chunk == j // chunk)


def attention(q, k, v, q_pos, scale, chunk, sink):
    """q [T, H, D] at positions q_pos, k [S, G, D], v [S, G, E] at positions 0..S-1 -> [T, H, E]. sink [H] or None."""
    T, H, _ = q.shape
    S, G, E = v.shape
    i, j = q_pos[:, None], torch.arange(S)[None]
    ok = j <= i
    if chunk:
        ok &= torch.div(i, chunk, rounding_mode="floor") == torch.div(j, chunk, rounding_mode="floor")
    out = torch.zeros(T, H, E, dtype=F)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~ok, -math.inf)
        top = s.max(-1).values
        if sink is not None:
            top = torch.maximum(top, sink[h].expand(T))
        e = torch.exp(s - top[:, None])
        den = e.sum(-1) + (torch.exp(sink[h] - top) if sink is not None else 0.0)
        out[:, h] = e @ v[:, g] / den[:, None]
    return out


def expert(x, up, down):
    return torch.relu(x @ up.T).square() @ down.T


def table_experts(x, ids, table, ups, downs):
    """Mean over the experts that the table names for each token id."""
    y = torch.zeros_like(x)
    for t, tok in enumerate(ids.tolist()):
        chosen = table[tok].tolist()
        y[t] = sum(expert(x[t], ups[e], downs[e]) for e in chosen) / len(chosen)
    return y


def loop_entry(x, x0, w):
    return torch.cat([x, x0], dim=-1) @ w.T


def schedule(cfg):
    """Layer numbers in execution order, with True where a pass over the looped range begins."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp or lp["start"] == lp["stop"]:
        return [(i, False) for i in range(n)]
    mid = [(i, i == lp["start"]) for _ in range(lp["times"]) for i in range(lp["start"], lp["stop"])]
    return [(i, False) for i in range(lp["start"])] + mid + [(i, False) for i in range(lp["stop"], n)]


def run(cfg, weights, tokens):
    """Whole sequence at once: (logits [T, vocab], residual stream after every layer run)."""
    W = {k: (t.to(F) if t.is_floating_point() else t.long()) for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.tensor(tokens)
    pos = torch.arange(len(tokens))
    norm = lambda x, n: layer_norm(x, W[n], W[n + ".b"], eps)   # noqa: E731
    x = x0 = W["embed"][ids]
    trail = []
    for i, enter in schedule(cfg):
        if enter:
            x = loop_entry(x, x0, W["loop.in"])
        m, f = cfg["layers"][i]["mixer"], cfg["layers"][i]["mlp"]
        h = norm(x, f"l{i}.norm1")
        q = (h @ W[f"l{i}.mix.q"].T).view(-1, m["heads"], m["dim"])
        k = (h @ W[f"l{i}.mix.k"].T).view(-1, m["kv_heads"], m["dim"])
        v = (h @ W[f"l{i}.mix.v"].T).view(-1, m["kv_heads"], m["vdim"])
        q, k = (rotate_pairs(t, pos, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
        a = attention(q, k, v, pos, m["scale"], m["mask"]["size"], W[f"l{i}.mix.sink"])
        x = x + norm(a.reshape(len(tokens), -1) @ W[f"l{i}.mix.o"].T, f"l{i}.norm1b")
        if f is not None:
            n = f["router"]["experts"]
            y = table_experts(norm(x, f"l{i}.norm2"), ids, W[f"l{i}.mlp.table"],
                              [W[f"l{i}.mlp.e{e}.up"] for e in range(n)], [W[f"l{i}.mlp.e{e}.down"] for e in range(n)])
            x = x + norm(y, f"l{i}.norm2b")
        trail.append(x)
    return norm(x, "final.norm") @ W["embed"].T * cfg["logit_scale"], trail


def greedy(cfg, weights, prompt, steps):
    """Greedy continuation and, per step, the gap between the best and the second-best logit."""
    toks, gaps = list(prompt), []
    for _ in range(steps):
        top = run(cfg, weights, toks)[0][-1].topk(2)
        toks.append(int(top.indices[0]))
        gaps.append(float(top.values[0] - top.values[1]))
    return toks[len(prompt):], gaps


# ---- small random models --------------------------------------------------------------------------------------------
def mixer(heads, kv_heads, dim, vdim, chunk, rot_dims, base, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
            "rot": {"dims": rot_dims, "base": base}, "scale": dim ** -0.5 if scale is None else scale}


def experts(n, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}


def config(layers, width, vocab, loop, eps=1e-5, logit_scale=1.0):
    return {"architecture": "Zobunex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "loop": loop, "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}


def model_a():
    """Every layer different: head counts and widths, q / k width unlike the v width, chunks, rotations, expert counts, a
    layer without a feed-forward; three passes over the middle."""
    return config([(mixer(6, 3, 64, 32, 37, 24, 500.0), experts(5, 3, 56)), (mixer(4, 1, 40, 72, 64, 40, 10000.0), None),
                   (mixer(2, 2, 128, 128, 50, 128, 3000.0, 0.07), experts(9, 1, 40)),
                   (mixer(8, 2, 16, 24, 101, 8, 777.0), experts(5, 3, 72))],
                  160, 321, {"start": 1, "stop": 3, "times": 3}, eps=1e-3, logit_scale=0.7)


def model_b():
    """Nothing a multiple of eight, one head each, one expert, the loop over all layers once."""
    return config([(mixer(3, 3, 20, 12, 16, 6, 100.0), experts(3, 2, 30)), (mixer(1, 1, 10, 18, 23, 10, 50.0), experts(1, 1, 13))],
                  90, 77, {"start": 0, "stop": 2, "times": 1}, eps=1e-2, logit_scale=1.3)


def model_c():
    """Heads wider than 128, more than sixteen query heads per key head, chunk 1 (a token sees itself only), no loop."""
    return config([(mixer(2, 1, 160, 136, 45, 160, 2000.0), experts(4, 4, 64)), (mixer(20, 1, 32, 32, 70, 32, 900.0), None),
                   (mixer(4, 4, 48, 56, 1, 48, 60.0), experts(33, 2, 24))], 200, 150, None, logit_scale=2.5)


def model_d():
    """Two layers with long chunks, for long contexts and the split-KV decode; loop at the start of the stack."""
    return config([(mixer(4, 2, 64, 64, 700, 32, 10000.0), experts(6, 2, 48)), (mixer(8, 1, 128, 96, 1000, 128, 5e5), experts(6, 2, 48))],
                  136, 200, {"start": 0, "stop": 1, "times": 2}, logit_scale=1.0)


MODELS = {"a": model_a, "b": model_b, "c": model_c, "d": model_d}


def random_weights(cfg, seed=0, peak=2.0):
    """bf16-representable weights; `peak` sets the spread of the attention scores."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, std=1.0):
        return (torch.randn(shape, generator=g) * std).to(torch.bfloat16)
    w = {"embed": rnd(V, W)}

    def norm(name):
        w[name] = (1.0 + 0.3 * torch.randn(W, generator=g)).to(torch.bfloat16)
        w[name + ".b"] = rnd(W, std=0.3)
    norm("final.norm")
    lp = cfg.get("loop")
    if lp and lp["start"] < lp["stop"]:
        w["loop.in"] = rnd(W, 2 * W, std=(2 * W) ** -0.5)
    for i, lay in enumerate(cfg["layers"]):
        m, f = lay["mixer"], lay["mlp"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            norm(f"l{i}.{n}")
        s = (peak / (m["scale"] * m["dim"] ** 0.5)) ** 0.5 * W ** -0.5
        w[f"l{i}.mix.q"] = rnd(m["heads"] * m["dim"], W, std=s)
        w[f"l{i}.mix.k"] = rnd(m["kv_heads"] * m["dim"], W, std=s)
        w[f"l{i}.mix.v"] = rnd(m["kv_heads"] * m["vdim"], W, std=W ** -0.5)
        w[f"l{i}.mix.sink"] = rnd(m["heads"], std=2.0)
        w[f"l{i}.mix.o"] = rnd(W, m["heads"] * m["vdim"], std=(m["heads"] * m["vdim"]) ** -0.5)
        if f:
            n, top, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
            w[f"l{i}.mlp.table"] = torch.stack([torch.randperm(n, generator=g)[:top] for _ in range(V)]).to(torch.int32)
            for e in range(n):
                w[f"l{i}.mlp.e{e}.up"] = rnd(ff, W, std=W ** -0.5)
                w[f"l{i}.mlp.e{e}.down"] = rnd(W, ff, std=ff ** -0.5)
    return w
