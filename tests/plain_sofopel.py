"""A plain, slow Sofopel decoder in numpy float64: one function per mechanism, whole sequences at once.

It shares no code with the library: the tests compare the library's logits and intermediate results with what these
functions give for the same configuration dict and the same tensors (name -> array).  Notation: T tokens, d the width,
H heads, G key/value heads; matrices are stored [out, in] and applied as x @ W.T.

`act` (everywhere optional) is applied to whatever a 16-bit run keeps in 16 bits between its steps: the identity here; a test
that passes small random changes learns how far roundings may move each position's logits (`shaken`).
"""
from __future__ import annotations

import math

import numpy as np


def exactly(a):
    return a


def shaken(seed, size=2.0 ** -8):
    """An `act` that changes every number by up to half of `size` of itself, as rounding to 8 significant bits does."""
    rng = np.random.default_rng(seed)
    return lambda a: a * (1.0 + size * (rng.random(np.shape(a)) - 0.5))


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def short_conv(u, w):
    """y[t, c] = sum_j w[c, j] u[t - taps + 1 + j, c], zeros before the start; u [T, channels], w [channels, taps]."""
    T, taps = u.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(padded[j:j + T] * w[:, j] for j in range(taps))


def frequencies(dims, base, scaling=None):
    """(the angle per position of every pair, what multiplies cosine and sine)."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            pair_of = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
            lo, hi = max(math.floor(pair_of(scaling["fast"])), 0), min(math.ceil(pair_of(scaling["slow"])), dims - 1)
            ramp = min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001)))
            f = ramp * f / scaling["factor"] + (1.0 - ramp) * f
        out.append(f)
    return np.array(out), (1.0 if scaling is None else 0.1 * math.log(scaling["factor"]) + 1.0)


def rotate(x, positions, rot, layout):
    """Turns the first rot["dims"] numbers of the last axis of x [T, ..., n] by the positions' angles."""
    if rot is None or rot["dims"] == 0:
        return x
    dims = rot["dims"]
    half = dims // 2
    freq, magnitude = frequencies(dims, rot["base"], rot.get("scaling"))
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]            # [T, half]
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (half,)
    c, s = magnitude * np.cos(ang).reshape(shape), magnitude * np.sin(ang).reshape(shape)
    out = x.copy()
    if layout == "half":
        a, b = x[..., :half], x[..., half:dims]
        out[..., :half], out[..., half:dims] = a * c - b * s, b * c + a * s
    else:                                                                            # neighbours (2i, 2i + 1)
        a, b = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = a * c - b * s, b * c + a * s
    return out


def same_chunk(T, size=None):
    """[T, T] booleans: query i sees key j <= i of its own chunk."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) if size is None else (j <= i) & (i // size == j // size)


def window_and_first(T, size=None, keep_first=0):
    """[T, T] booleans: query i sees key j <= i inside the window or among the first positions."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) if size is None else (j <= i) & ((i - j < size) | (j < keep_first))


def softmax(s):
    p = np.exp(s - s.max(axis=1, keepdims=True))
    return p / p.sum(axis=1, keepdims=True)


def softmax_plus_one(s):
    """Rows of scores (-inf where hidden) to weights with one more in the denominator: a sink of score 0 without a value."""
    top = np.maximum(s.max(axis=1, keepdims=True), 0.0)
    p = np.exp(s - top)
    return p / (p.sum(axis=1, keepdims=True) + np.exp(-top))


def map_weight(W, pre, diff):
    """lambda: how much of the second map is taken off the first."""
    return np.exp(W[pre + "lq1"] @ W[pre + "lk1"]) - np.exp(W[pre + "lq2"] @ W[pre + "lk2"]) + diff


def difference_of_maps(a1, a2, lam, diff, eps):
    """[..., vdim] outputs of the two maps to one head's output."""
    return rms_unit(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, positions, W, pre, m, eps, act=exactly):
    T, H, G, n, mv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (act(h @ W[pre + t].T) for t in "qkv")
    if m.get("conv"):
        q, k, v = (short_conv(x, W[pre + t + ".conv"]) for x, t in ((q, "q"), (k, "k"), (v, "v")))
    q = act(rotate(q.reshape(T, H, 2, n), positions, m.get("rot"), "adjacent"))
    k = act(rotate(k.reshape(T, G, 2, n), positions, m.get("rot"), "adjacent"))
    v = act(v).reshape(T, G, mv)
    mask = same_chunk(T, m["mask"]["size"] if m.get("mask") else None)
    lam = map_weight(W, pre, m["diff"])
    out = np.zeros((T, H, mv))
    for a in range(H):
        g = a // (H // G)
        maps = [act(softmax(np.where(mask, q[:, a, j] @ k[:, g, j].T * m["scale"], -np.inf)) @ v[:, g]) for j in range(2)]
        out[:, a] = difference_of_maps(maps[0], maps[1], lam, m["diff"], eps)
    return act(out).reshape(T, H * mv) @ W[pre + "o"].T


def windowed_attention(h, positions, W, pre, m, eps, act=exactly):
    T, H, G, n, mv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (act(h @ W[pre + t].T) for t in "qkv")
    q = act(rotate(rms_unit(q.reshape(T, H, n), eps) * W[pre + "q.norm"], positions, m.get("rot"), "half"))
    k = act(rotate(rms_unit(k.reshape(T, G, n), eps) * W[pre + "k.norm"], positions, m.get("rot"), "half"))
    v = v.reshape(T, G, mv)
    mk = m.get("mask")
    mask = window_and_first(T, mk["size"], mk.get("keep_first", 0)) if mk else window_and_first(T)
    out = np.zeros((T, H, mv))
    for a in range(H):
        g = a // (H // G)
        out[:, a] = softmax_plus_one(np.where(mask, q[:, a] @ k[:, g].T * m["scale"], -np.inf)) @ v[:, g]
    out = act(act(out) * sigmoid(h @ W[pre + "g"].T)[:, :, None])
    return out.reshape(T, H * mv) @ W[pre + "o"].T


def decays(h, W, pre, tau, act=exactly):
    """alpha [T, heads * dim] = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)."""
    z = act(h @ W[pre + "a1"].T) @ W[pre + "a2"].T + W[pre + "a2.b"]
    return np.exp(-np.logaddexp(0.0, -z) / tau)


def gated_linear_attention(h, W, pre, m, eps, state=None, act=exactly):
    """`state` [H, n, mv] is carried in and returned."""
    T, H, n, mv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = act(h @ W[pre + "q"].T).reshape(T, H, n) * n ** -0.5
    k = act(h @ W[pre + "k"].T).reshape(T, H, n)
    v = act(h @ W[pre + "v"].T).reshape(T, H, mv)
    alpha = decays(h, W, pre, m["tau"], act).reshape(T, H, n)
    S = np.zeros((H, n, mv)) if state is None else state.copy()
    o = np.zeros((T, H, mv))
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hnm,hn->hm", S, q[t])
    g = act(h @ W[pre + "g"].T)
    o = act((rms_unit(o, eps) * W[pre + "norm"]).reshape(T, H * mv) * (g * sigmoid(g)))
    return o @ W[pre + "o"].T, S


def clamped_gated_mlp(h, W, pre, limit, act=exactly):
    g, u = np.minimum(h @ W[pre + "gate"].T, limit), np.clip(h @ W[pre + "up"].T, -limit, limit)
    return act(g * sigmoid(1.702 * g) * (u + 1.0)) @ W[pre + "down"].T


def runs(cfg):
    """The layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


def layer(x, i, cfg, W, positions, act=exactly):
    """Both sublayers read one norm of the stream, and their sum joins it."""
    lp, lay, eps = f"l{i}.", cfg["layers"][i], cfg["norm"]["eps"]
    h = act(rms_unit(x, eps) * W[lp + "norm1"])
    m = lay["mixer"]
    if lay["type"] == "gla":
        y = gated_linear_attention(h, W, lp + "mix.", m, eps, act=act)[0]
    elif lay["type"] == "attention":
        y = differential_attention(h, positions, W, lp + "mix.", m, eps, act)
    else:
        y = windowed_attention(h, positions, W, lp + "mix.", m, eps, act)
    if lay.get("mlp") is not None:
        y = y + clamped_gated_mlp(h, W, lp + "mlp.", lay["mlp"]["limit"], act)
    return x + cfg["residual_mult"] * y


def forward(cfg, W, tokens, return_layers=False, act=exactly):
    """Logits [T, vocab] of one sequence from its first token (float64); optionally the stream after every layer run."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    positions = np.arange(len(tokens))
    x, after = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"], []
    for i in runs(cfg):
        x = layer(x, i, cfg, W, positions, act)
        after.append(x)
    logits = act(rms_unit(x, cfg["norm"]["eps"]) * W["final.norm"]) @ W["head"].T
    return (logits, np.stack(after)) if return_layers else logits


def bf16_values(a):
    """Rounds to the nearest bfloat16 value (ties to even), kept as float64: a bfloat16 file then holds the weights exactly."""
    f = np.ascontiguousarray(np.asarray(a, dtype=np.float32))
    u = f.view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32)
    return u.view(np.float32).astype(np.float64).reshape(np.shape(a))


def random_weights(cfg, seed=0, rank=None):
    """Weights for `cfg` (name -> float64 array of bfloat16 values).  `rank`: the width between the decay's two matrices, by
    layer (a dict), or one for all."""
    rng = np.random.default_rng(seed)
    d, out = int(cfg["width"]), {}

    def put(name, shape, std=None, mean=0.0):
        std = std if std is not None else (1.0 / math.sqrt(shape[-1]) if len(shape) > 1 else 0.5)
        out[name] = bf16_values(rng.standard_normal(shape) * std + mean)

    put("embed", (int(cfg["vocab"]), d), 1.0 / max(1.0, float(cfg["embedding"]["scale"])))
    put("final.norm", (d,), 0.1, 1.0)
    put("head", (int(cfg["vocab"]), d))
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        x = p + "mix."
        put(p + "norm1", (d,), 0.1, 1.0)
        if lay.get("mlp") is not None:
            ff = int(lay["mlp"]["ff"])
            put(p + "mlp.gate", (ff, d), 2.0 / math.sqrt(d)); put(p + "mlp.up", (ff, d), 2.0 / math.sqrt(d)); put(p + "mlp.down", (d, ff))
        H, n, mv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        G = int(m.get("kv_heads", H))
        put(x + "o", (d, H * mv), 2.0 / math.sqrt(H * mv))
        if lay["type"] == "gla":
            r = rank.get(i, 4) if isinstance(rank, dict) else (rank or 4)
            put(x + "q", (H * n, d)); put(x + "k", (H * n, d)); put(x + "v", (H * mv, d)); put(x + "g", (H * mv, d), 2.0 / math.sqrt(d))
            put(x + "a1", (r, d), 2.0 / math.sqrt(d)); put(x + "a2", (H * n, r), 1.0 / math.sqrt(r)); put(x + "a2.b", (H * n,), 1.0, 1.0)
            put(x + "norm", (mv,), 0.2, 1.0)
        elif lay["type"] == "attention":
            put(x + "q", (H * 2 * n, d), 2.0 / math.sqrt(d)); put(x + "k", (G * 2 * n, d), 2.0 / math.sqrt(d)); put(x + "v", (G * mv, d))
            if m.get("conv"):
                for t, c in (("q", H * 2 * n), ("k", G * 2 * n), ("v", G * mv)):
                    put(x + t + ".conv", (c, int(m["conv"])), 0.6)
            for t in ("lq1", "lk1", "lq2", "lk2"):
                put(x + t, (n,), 0.6 / n ** 0.25)
        else:
            put(x + "q", (H * n, d)); put(x + "k", (G * n, d)); put(x + "v", (G * mv, d))
            put(x + "q.norm", (n,), 0.3, 1.5); put(x + "k.norm", (n,), 0.3, 1.5); put(x + "g", (H, d), 2.0 / math.sqrt(d))
    return out
