"""Plain restatement of the Kuvelix decoder, one function per mechanism, in float64, position by position, without any cache.

Nothing here is shared with the engine: the tests compare the engine's kernels, caches and schedules with these loops.
A model is (cfg, w): `cfg` the dictionary of config.json, `w` a dictionary name -> numpy array with the checkpoint's names
(`embed`, `embed.norm`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`).

The design: x = rms_w(embed[token]); a layer is PARALLEL with one norm, u = rms_w(x), x += mixer(u) + ff(u); a block of layers may
run several times in a row with the same tensors and nothing in between; norm and tied head at the end. The mixer is grouped
attention with biased projections, a weighted norm of every q / k head, interleaved rotary pairs (frequencies optionally divided by a
constant), plain causal softmax and a sigmoid output gate per channel. Feed-forwards: W_down(gelu_tanh(W_gate u) * W_up u), or a
mixture of bounded gated experts behind a softmax router whose choice (not its weights) carries a correction, with expert groups and
with identity experts that hand u on.

Notation: h is a sublayer's input [T, width]; every Linear weight is [out, in] and applied as h @ W.T; t, i, j are positions
of one sequence, counted from 0.
"""
import math

import numpy as np

F = np.float64


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * np.asarray(weight, F)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------------- rotations
def rotary_frequencies(rot):
    """Angle per position of every rotated pair; `scaling.factor` slows all of them down alike."""
    dims, base = int(rot["dims"]), float(rot["base"])
    factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    return np.array([base ** (-2.0 * i / dims) / factor for i in range(dims // 2)], F)


def rotate_pairs(x, pos, freq):
    """Turns the pairs (2i, 2i + 1), i < len(freq), of x's last axis by pos * freq_i; the rest passes. pos a number."""
    n = 2 * len(freq)
    out = np.array(x, F, copy=True)
    c, s = np.cos(pos * freq), np.sin(pos * freq)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------- attention
def project(h, p, name):
    """W h + b."""
    return h @ p[name].T + p[name + ".b"]


def queries_keys_values(h, p, mix, eps):
    """q [T, H, dim], k [T, G, dim] normed per head and turned by their position, v [T, G, vdim]."""
    T = h.shape[0]
    H, G, dk, dv = (int(mix[n]) for n in ("heads", "kv_heads", "dim", "vdim"))
    q = rms_norm(project(h, p, "q").reshape(T, H, dk), p["q.norm"], eps)
    k = rms_norm(project(h, p, "k").reshape(T, G, dk), p["k.norm"], eps)
    v = project(h, p, "v").reshape(T, G, dv)
    if mix.get("rot"):
        freq = rotary_frequencies(mix["rot"])
        q = np.stack([rotate_pairs(q[t], t, freq) for t in range(T)])
        k = np.stack([rotate_pairs(k[t], t, freq) for t in range(T)])
    return q, k, v


def softmax_attend(scores, values):
    e = np.exp(scores - scores.max())
    return (e / e.sum()) @ values


def attention(h, p, mix, eps):
    T = h.shape[0]
    H, G, dv, scale = int(mix["heads"]), int(mix["kv_heads"]), int(mix["vdim"]), float(mix["scale"])
    q, k, v = queries_keys_values(h, p, mix, eps)
    out = np.zeros((T, H, dv), F)
    for i in range(T):
        for a in range(H):
            g = a // (H // G)
            out[i, a] = softmax_attend(k[:i + 1, g] @ q[i, a] * scale, v[:i + 1, g])
    gate = sigmoid(h @ p["g"].T)
    return (out.reshape(T, H * dv) * gate) @ p["o"].T


# ------------------------------------------------------------------------------------------------- feed-forwards
def dense_ff(h, p):
    return (gelu_tanh(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def expert(h, gate, up, down, limit):
    """W_down (g sigmoid(1.702 g) (u + 1)), g = min(W_gate h, limit), u = W_up h held to +-limit (limit None: unbounded)."""
    g, u = h @ gate.T, h @ up.T
    if limit is not None:
        g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, router_w, correction, r):
    """Chosen experts and their weights for every row. Scores: softmax over every router row (identity experts last). What is compared
    is score + correction: groups of neighbours count by their best, the best `keep` groups compete, the `top` largest win. The
    weights are the winners' scores without the correction, over their sum."""
    top = int(r["top"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    G, keep = int(groups["count"]), int(groups["keep"])
    z = h @ router_w.T
    s = np.exp(z - z.max(-1, keepdims=True))
    s = s / s.sum(-1, keepdims=True)
    E = s.shape[1]
    c = s + np.asarray(correction, F)
    idx, wgt = [], []
    for t in range(h.shape[0]):
        gs = c[t].reshape(G, E // G).max(-1)
        alive = sorted(range(G), key=lambda g: (-gs[g], g))[:keep]
        cand = [e for e in range(E) if e // (E // G) in alive]
        chosen = sorted(cand, key=lambda e: (-c[t, e], e))[:top]
        total = sum(s[t, e] for e in chosen) + 1e-20
        idx.append(chosen)
        wgt.append([s[t, e] / total for e in chosen])
    return idx, wgt


def moe_ff(h, p, mlp):
    real, limit = int(mlp["router"]["experts"]), mlp["expert"].get("limit")
    idx, wgt = route(h, p["router"], p["correction"], mlp["router"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(idx[t], wgt[t]):
            out[t] += g * (h[t] if e >= real else expert(h[t:t + 1], p[f"e{e}.gate"], p[f"e{e}.up"], p[f"e{e}.down"], limit)[0])
    return out


def feed_forward(h, p, mlp):
    return moe_ff(h, p, mlp) if mlp["kind"] == "moe" else dense_ff(h, p)


# ------------------------------------------------------------------------------------------------- the model
def layer_params(w, i, part):
    pre = f"l{i}.{part}."
    return {k[len(pre):]: np.asarray(v, F) for k, v in w.items() if k.startswith(pre)}


def layer_order(cfg):
    """Layers in the order they run; a looped block appears once per pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b, t = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return list(range(a)) + list(range(a, b)) * t + list(range(b, n))


def embedding(cfg, w, tokens):
    return rms_norm(np.asarray(w["embed"], F)[list(tokens)], w["embed.norm"], float(cfg["norm"]["eps"]))


def layer_step(x, w, i, layer, eps):
    """x + mixer(u) + ff(u), u = rms_w(x): both sublayers read the same normed input."""
    u = rms_norm(x, w[f"l{i}.norm1"], eps)
    y = attention(u, layer_params(w, i, "mix"), layer["mixer"], eps)
    if layer.get("mlp"):
        y = y + feed_forward(u, layer_params(w, i, "mlp"), layer["mlp"])
    return x + y


def forward(cfg, w, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer run)."""
    eps = float(cfg["norm"]["eps"])
    x = embedding(cfg, w, tokens)
    per_layer = []
    for i in layer_order(cfg):
        x = layer_step(x, w, i, cfg["layers"][i], eps)
        per_layer.append(x.copy())
    logits = rms_norm(x, w["final.norm"], eps) @ np.asarray(w["embed"], F).T
    return (logits, np.stack(per_layer)) if return_layers else logits


def bf16_round(a):
    """Round float32 values to the nearest bfloat16 (ties to even), returned as float32."""
    u = np.asarray(a, np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32)


def tensor_shapes(cfg):
    """name -> shape of every tensor a checkpoint of this configuration holds."""
    width, vocab = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": (vocab, width), "embed.norm": (width,), "final.norm": (width,)}
    for i, layer in enumerate(cfg["layers"]):
        mix, mlp, a = layer["mixer"], layer.get("mlp"), f"l{i}."
        out[a + "norm1"] = (width,)
        H, G, dk, dv = (int(mix[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            out[a + "mix." + n], out[a + "mix." + n + ".b"] = (rows, width), (rows,)
        out[a + "mix.q.norm"] = out[a + "mix.k.norm"] = (dk,)
        out[a + "mix.g"], out[a + "mix.o"] = (H * dv, width), (width, H * dv)
        if mlp and mlp["kind"] == "moe":
            r, ff = mlp["router"], int(mlp["expert"]["ff"])
            n = int(r["experts"]) + int(r.get("identity", 0) or 0)
            out[a + "mlp.router"], out[a + "mlp.correction"] = (n, width), (n,)
            for e in range(int(r["experts"])):
                out[a + f"mlp.e{e}.gate"] = out[a + f"mlp.e{e}.up"] = (ff, width)
                out[a + f"mlp.e{e}.down"] = (width, ff)
        elif mlp:
            ff = int(mlp["ff"])
            out[a + "mlp.gate"] = out[a + "mlp.up"] = (ff, width)
            out[a + "mlp.down"] = (width, ff)
    return out


def random_weights(cfg, seed=0, gain=1.0):
    """Random tensors (values exactly representable in bfloat16) for any configuration: Linear weights ~ N(0, gain^2 / in), norm
    weights near 1, biases ~ N(0, 0.5^2), corrections of the size of a score in either sign, the embedding's rows longer than 1 and the
    head (the same table) with logits of order 1 after the norms."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf == "correction":
            t = 1.5 * rng.standard_normal(shape) / shape[0]
        elif leaf == "b":
            t = 0.5 * rng.standard_normal(shape)
        elif len(shape) == 1:
            t = 1.0 + 0.2 * rng.standard_normal(shape)
        elif leaf == "embed":
            t = 1.5 * rng.standard_normal(shape) / math.sqrt(shape[1])
        elif leaf == "router":
            t = 2.0 * rng.standard_normal(shape) / math.sqrt(shape[1])
        else:
            t = gain * rng.standard_normal(shape) / math.sqrt(shape[1])
        w[name] = bf16_round(t.astype(np.float32))
    return w
