"""Plain restatement of the Ramosun decoder, one function per mechanism, in float64, position by position, without any cache.

Nothing here is shared with the engine: the tests compare the engine's kernels, caches and schedules with these loops.
A model is (cfg, w): `cfg` the dictionary of config.json, `w` a dictionary name -> numpy array with the checkpoint's names
(`embed`, `loop.in`, `l<i>.norm1[.alpha|.b]`, `l<i>.norm2[...]`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm[...]`).

The design: x = embed[token] (x0); a layer is PARALLEL with a norm for each sublayer, x += mixer(N1(x)) + ff(N2(x)), both norms of
the same x; the norm is a dynamic tanh, N(x) = tanh(alpha x) w + b, which computes no statistics. A block of layers may run several
times in a row with the same tensors; in front of every pass x becomes W_in [x; x0]. Norm, tied head, soft-capped logits at the end.
Mixers: `mlstm` (matrix memory with exponential gates under a running maximum), `delta` (gated delta rule behind a short convolution)
and `attention` (grouped heads whose values are the raw keys, a norm over the whole q / k projection, rotate-half positions with
wavelength-banded frequency scaling, a sliding window, a learned sink per head). Feed-forward: W_down gelu(W_up h).

Notation: h is a sublayer's input [T, width]; every Linear weight is [out, in] and applied as h @ W.T; t, i, j are positions
of one sequence, counted from 0.
"""
import math

import numpy as np

F = np.float64


def dyt(x, w, name):
    """Dynamic tanh `name` of w: tanh(alpha x) * weight + bias, element by element."""
    alpha = float(np.asarray(w[name + ".alpha"], F).reshape(()))
    return np.tanh(alpha * x) * np.asarray(w[name], F) + np.asarray(w[name + ".b"], F)


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def softplus(z):
    return np.logaddexp(0.0, z)


_erf = np.frompyfunc(math.erf, 1, 1)


def gelu(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)).astype(F))


# ------------------------------------------------------------------------------------------------- convolution over time
def causal_conv(u, taps_w):
    """y_t = sum_j w[:, j] * u_(t - taps + 1 + j) per channel, zeros in front of the sequence. u [T, C], taps_w [C, taps]."""
    T, C = u.shape
    taps = taps_w.shape[1]
    y = np.zeros((T, C), F)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += taps_w[:, j] * u[s]
    return y


# ------------------------------------------------------------------------------------------------- rotations
def rotary_frequencies(rot):
    """Angle per position of every rotated pair. With `scaling` a pair whose wavelength 2 pi / f is below original / high keeps its
    frequency, one above original / low is slowed down by factor, and the ones between are blended linearly in original / wavelength."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc:
        factor, low, high, orig = (float(sc[k]) for k in ("factor", "low", "high", "original"))
        for i, fi in enumerate(f):
            wave = 2.0 * math.pi / fi
            if wave < orig / high:
                continue
            if wave > orig / low:
                f[i] = fi / factor
            else:
                s = (orig / wave - low) / (high - low)
                f[i] = (1.0 - s) * fi / factor + s * fi
    return np.array(f, F)


def rotate_half(x, pos, freq):
    """Turns the pairs (m, m + n) of the leading 2n entries of x's last axis by pos * freq_m, n = len(freq); the rest passes."""
    n = len(freq)
    out = np.array(x, F, copy=True)
    c, s = np.cos(pos * freq), np.sin(pos * freq)
    u, v = x[..., 0:n], x[..., n:2 * n]
    out[..., 0:n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------- visibility and softmax
def sees_window(i, j, size):
    """The last `size` positions, the query's own included (size None: plain causal)."""
    return j <= i and (size is None or i - j < size)


def softmax_attend(scores, values, sink):
    """Weights exp(s_j) / (sum exp(s) + exp(sink)) over the given keys, applied to their values (sink None: no extra term)."""
    m = scores.max() if sink is None else max(scores.max(), sink)
    e = np.exp(scores - m)
    den = e.sum() + (0.0 if sink is None else math.exp(sink - m))
    return (e / den) @ values


# ------------------------------------------------------------------------------------------------- mixers
def mlstm_gates(h, p, mix):
    """Log input and log forget gate, [T, heads] each."""
    cap = float(mix["gate_cap"])
    i = cap * np.tanh((h @ p["i"].T + p["i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh((h @ p["f"].T + p["f.b"]) / cap))
    return i, f


def mlstm_memory(q, k, v, i, f):
    """One head: q, k [T, dim] (q scaled), v [T, vdim], log gates i, f [T] -> read-outs [T, vdim]."""
    T, dk = q.shape
    S, n, m = np.zeros((dk, v.shape[1]), F), np.zeros(dk, F), 0.0
    out = np.zeros_like(v)
    for t in range(T):
        m_new = max(f[t] + m, i[t])
        keep, write = math.exp(f[t] + m - m_new), math.exp(i[t] - m_new)
        S = keep * S + write * np.outer(k[t], v[t])
        n = keep * n + write * k[t]
        m = m_new
        out[t] = (S.T @ q[t]) / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6)
    return out


def mlstm(h, p, mix, eps):
    H, dk, dv = int(mix["heads"]), int(mix["dim"]), int(mix["vdim"])
    T = h.shape[0]
    q = (h @ p["q"].T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ p["k"].T).reshape(T, H, dk)
    v = (h @ p["v"].T).reshape(T, H, dv)
    i, f = mlstm_gates(h, p, mix)
    o = np.stack([mlstm_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]) for a in range(H)], axis=1)
    y = rms_unit(o, eps).reshape(T, H * dv) * p["norm"]
    return (y * sigmoid(h @ p["g"].T)) @ p["o"].T


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def delta_memory(q, k, v, beta, g):
    """One head: unit q (scaled) and k [T, dim], v [T, vdim], write strength beta and decay g [T] -> read-outs [T, vdim]."""
    S = np.zeros((q.shape[1], v.shape[1]), F)
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out


def delta(h, p, mix, eps):
    H, G, dk, dv = int(mix["heads"]), int(mix["kv_heads"]), int(mix["dim"]), int(mix["vdim"])
    T = h.shape[0]
    q, k, v = (silu(causal_conv(h @ p[n].T, p[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, G, dk)) * dk ** -0.5
    k = unit(k.reshape(T, G, dk))
    v = v.reshape(T, H, dv)
    beta = sigmoid(h @ p["b"].T)
    g = np.exp(-np.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))
    o = np.stack([delta_memory(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], beta[:, a], g[:, a]) for a in range(H)], axis=1)
    y = rms_unit(o, eps) * p["norm"] * silu(h @ p["g"].T).reshape(T, H, dv)
    return y.reshape(T, H * dv) @ p["o"].T


def attention(h, p, mix, eps):
    H, G, dk = int(mix["heads"]), int(mix["kv_heads"]), int(mix["dim"])
    T = h.shape[0]
    raw = h @ p["k"].T
    v = raw.reshape(T, G, dk)                                            # the values are the keys as projected
    q = (rms_unit(h @ p["q"].T, eps) * p["q.norm"]).reshape(T, H, dk)      # one norm over all heads together
    k = (rms_unit(raw, eps) * p["k.norm"]).reshape(T, G, dk)
    rot = mix.get("rot")
    if rot:
        f = rotary_frequencies(rot)
        q = np.stack([rotate_half(q[t], t, f) for t in range(T)])
        k = np.stack([rotate_half(k[t], t, f) for t in range(T)])
    size, scale = (mix.get("mask") or {}).get("size"), float(mix["scale"])
    out = np.zeros((T, H, dk), F)
    for i in range(T):
        js = [j for j in range(i + 1) if sees_window(i, j, size)]
        for a in range(H):
            g = a // (H // G)
            out[i, a] = softmax_attend(k[js, g] @ q[i, a] * scale, v[js, g], float(p["sink"][a]))
    return out.reshape(T, H * dk) @ p["o"].T


MIXERS = {"mlstm": mlstm, "delta": delta, "attention": attention}


# ------------------------------------------------------------------------------------------------- feed-forward
def feed_forward(h, p):
    return gelu(h @ p["up"].T) @ p["down"].T


# ------------------------------------------------------------------------------------------------- the model
def layer_params(w, i, part):
    pre = f"l{i}.{part}."
    return {k[len(pre):]: np.asarray(v, F) for k, v in w.items() if k.startswith(pre)}


def layer_order(cfg):
    """[(layer, whether its run opens a pass of the looped block)] in the order of execution."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return [(i, False) for i in range(a)] + [(i, i == a) for i in range(a, b)] * times + [(i, False) for i in range(b, n)]


def open_pass(x, x0, w):
    return np.concatenate([x, x0], axis=-1) @ np.asarray(w["loop.in"], F).T


def layer_step(x, cfg, w, i):
    """x after layer i."""
    layer, eps = cfg["layers"][i], float(cfg["norm"]["eps"])
    y = MIXERS[layer["type"]](dyt(x, w, f"l{i}.norm1"), layer_params(w, i, "mix"), layer["mixer"], eps)
    if layer.get("mlp"):
        if layer["mlp"].get("kind", "dense") != "dense":
            raise NotImplementedError(layer["mlp"]["kind"])
        y = y + feed_forward(dyt(x, w, f"l{i}.norm2"), layer_params(w, i, "mlp"))
    return x + y


def head(x, cfg, w):
    logits = dyt(x, w, "final.norm") @ np.asarray(w["embed"], F).T
    cap = float(cfg.get("logit_softcap") or 0.0)
    return cap * np.tanh(logits / cap) if cap > 0 else logits


def forward(cfg, w, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer run)."""
    x0 = np.asarray(w["embed"], F)[np.asarray(tokens)]
    x, layers = x0, []
    for i, opens in layer_order(cfg):
        if opens:
            x = open_pass(x, x0, w)
        x = layer_step(x, cfg, w, i)
        layers.append(x.copy())
    logits = head(x, cfg, w)
    return (logits, np.stack(layers)) if return_layers else logits


# ------------------------------------------------------------------------------------------------- random models
def bf16_round(a):
    """Nearest bfloat16 (ties to even) of float32 values, returned as float32."""
    b = np.asarray(a, np.float32).view(np.uint32).astype(np.uint64)
    b = ((b + 0x7FFF + ((b >> 16) & 1)) >> 16) << 16
    return b.astype(np.uint32).view(np.float32)


def tensor_shapes(cfg):
    """name -> shape of every tensor of a model of this configuration."""
    W, V = int(cfg["width"]), int(cfg["vocab"])
    s = {"embed": (V, W)}

    def norm(name):
        s.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})

    norm("final.norm")
    if cfg.get("loop"):
        s["loop.in"] = (W, 2 * W)
    for i, layer in enumerate(cfg["layers"]):
        mix, t, pre = layer["mixer"], layer["type"], f"l{i}.mix."
        norm(f"l{i}.norm1")
        H, dk = int(mix["heads"]), int(mix["dim"])
        dv = int(mix.get("vdim", dk))
        s[pre + "o"] = (W, H * dv)
        if t == "mlstm":
            s.update({pre + "q": (H * dk, W), pre + "k": (H * dk, W), pre + "v": (H * dv, W), pre + "g": (H * dv, W), pre + "norm": (H * dv,),
                      pre + "i": (H, W), pre + "i.b": (H,), pre + "f": (H, W), pre + "f.b": (H,)})
        elif t == "delta":
            G, taps = int(mix["kv_heads"]), int(mix["conv"])
            for n, c in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                s.update({pre + n: (c, W), pre + n + ".conv": (c, taps)})
            s.update({pre + "b": (H, W), pre + "a": (H, W), pre + "A_log": (H,), pre + "dt_bias": (H,), pre + "g": (H * dv, W), pre + "norm": (dv,)})
        elif t == "attention":
            G = int(mix["kv_heads"])
            s.update({pre + "q": (H * dk, W), pre + "k": (G * dk, W), pre + "q.norm": (H * dk,), pre + "k.norm": (G * dk,), pre + "sink": (H,)})
        else:
            raise NotImplementedError(t)
        if layer.get("mlp"):
            ff = int(layer["mlp"]["ff"])
            norm(f"l{i}.norm2")
            s.update({f"l{i}.mlp.up": (ff, W), f"l{i}.mlp.down": (W, ff)})
    return s


def random_weights(cfg, seed=0, gain=1.0):
    """Random bfloat16-representable tensors: matrices ~ N(0, gain^2 / fan_in), norm weights near 1 with small biases and slopes between
    0.4 and 1.2, gate biases that spread memories between short and long."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf == "alpha":
            a = rng.uniform(0.4, 1.2, shape)
        elif leaf in ("norm1", "norm2", "norm") :
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name.endswith(".i.b"):
            a = rng.uniform(-3.0, 2.0, shape)
        elif name.endswith(".f.b"):
            a = rng.uniform(0.0, 6.0, shape)
        elif leaf == "b" and "norm" in name:
            a = 0.1 * rng.standard_normal(shape)
        elif leaf == "A_log":
            a = rng.uniform(-1.5, 1.0, shape)
        elif leaf == "dt_bias":
            a = rng.uniform(-4.0, 0.5, shape)
        elif leaf == "sink":
            a = rng.standard_normal(shape)
        elif leaf == "conv":
            a = 0.6 * rng.standard_normal(shape)
        elif name == "embed":
            a = rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) * gain / math.sqrt(shape[-1])
        w[name] = bf16_round(np.asarray(a, np.float32).reshape(shape))
    return w
