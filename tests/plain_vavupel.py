"""A plain, slow Vavupel decoder in numpy float64: one function per mechanism, whole sequences at once.

It shares no code with the library: the tests compare the library's logits and intermediate results with what these
functions give for the same configuration dict and the same tensors (name -> array).  Notation: T tokens, d the width,
H heads; matrices are stored [out, in] and applied as x @ W.T.

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


def tanh_norm(x, W, name):
    """tanh(alpha x) * w + b, element by element."""
    return np.tanh(float(np.reshape(W[name + ".alpha"], ())) * x) * W[name] + W[name + ".b"]


def bigram_rows(tokens, spec):
    """Rows of the pair table: one per (previous token, token), the extra last row for a sequence's first token."""
    rows = np.zeros(len(tokens), dtype=np.int64)
    for t, tok in enumerate(tokens):
        rows[t] = spec["buckets"] if t == 0 else (int(tokens[t - 1]) * spec["mul_prev"] + int(tok) * spec["mul_cur"]) % spec["buckets"]
    return rows


def embedded(tokens, cfg, W):
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    spec = cfg["embedding"].get("bigram")
    if spec is not None:
        x = x + W["bigram"][bigram_rows(tokens, spec)]
    return tanh_norm(x, W, "embed.norm")


def rotate(x, positions, dims, base, layout):
    """Turns the first `dims` numbers of the last axis of x [T, ..., n] by the positions' angles."""
    if dims == 0:
        return x
    half = dims // 2
    freq = base ** (-2.0 * np.arange(half) / dims)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]            # [T, half]
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (half,)
    c, s = np.cos(ang).reshape(shape), np.sin(ang).reshape(shape)
    out = x.copy()
    if layout == "half":
        a, b = x[..., :half], x[..., half:dims]
        out[..., :half], out[..., half:dims] = a * c - b * s, b * c + a * s
    else:                                                                            # neighbours (2i, 2i + 1)
        a, b = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = a * c - b * s, b * c + a * s
    return out


def visible(T, size=None):
    """[T, T] booleans: query i sees key j."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) if size is None else (j <= i) & (i - j < size)


def softmax_with_sink(s, sink):
    """Rows of scores [T, T] (-inf where hidden) to weights; exp(sink) joins the denominator alone."""
    top = np.maximum(s.max(axis=1, keepdims=True), sink)
    p = np.exp(s - top)
    return p / (p.sum(axis=1, keepdims=True) + np.exp(sink - top))


def latent_attention(h, positions, W, pre, m, eps, act=exactly):
    T, H, n, r, mv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = act(h @ W[pre + "q"].T).reshape(T, H, n + r)
    down = act(h @ W[pre + "dkv"].T)
    c = act(rms_unit(down[:, :rank], eps) * W[pre + "dkv.norm"])
    k_rot = act(rotate(down[:, rank:], positions, m["rot"]["dims"], m["rot"]["base"], "adjacent"))   # [T, r], all heads share it
    q_rot = act(rotate(q[:, :, n:], positions, m["rot"]["dims"], m["rot"]["base"], "adjacent"))
    k = (c @ W[pre + "uk"].T).reshape(T, H, n)
    v = (c @ W[pre + "uv"].T).reshape(T, H, mv)
    mask = visible(T, m["mask"]["size"] if m.get("mask") else None)
    out = np.zeros((T, H, mv))
    for a in range(H):
        s = (q[:, a, :n] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]
        out[:, a] = softmax_with_sink(np.where(mask, s, -np.inf), float(W[pre + "sink"][a])) @ v[:, a]
    out = act(act(out) * sigmoid(act(h @ W[pre + "g"].T))[:, :, None])
    return out.reshape(T, H * mv) @ W[pre + "o"].T


def retention(h, positions, W, pre, m, eps, state=None, act=exactly):
    """Linear attention with a constant decay per head.  `state` [H, n, mv] is carried in and returned."""
    T, H, n, mv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate(act(h @ W[pre + "q"].T).reshape(T, H, n), positions, m["rot"]["dims"], m["rot"]["base"], "half")
    k = rotate(act(h @ W[pre + "k"].T).reshape(T, H, n), positions, m["rot"]["dims"], m["rot"]["base"], "half") * n ** -0.5
    v = act(h @ W[pre + "v"].T).reshape(T, H, mv)
    S = np.zeros((H, n, mv)) if state is None else state.copy()
    decay = np.asarray(m["decay"], dtype=np.float64)[:, None, None]
    o = np.zeros((T, H, mv))
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hnm,hn->hm", S, q[t])
    g = act(h @ W[pre + "g"].T)
    o = act(rms_unit(o, eps).reshape(T, H * mv) * (g * sigmoid(g)))
    return o @ W[pre + "o"].T, S


def squared_relu_mlp(h, W, pre, act=exactly):
    return act(np.maximum(h @ W[pre + "up"].T, 0.0) ** 2) @ W[pre + "down"].T


def injected(x, x0, W, act=exactly):
    """What a pass over the looped layers starts from: a product of the stream beside the embedding output."""
    return act(np.concatenate([x, x0], axis=1)) @ W["loop.in"].T


def softcap(z, cap):
    return z if not cap else cap * np.tanh(z / cap)


def runs(cfg):
    """The layers in the order they run, each with whether a pass over the loop starts right before it."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    body = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return [(i, False) for i in range(loop["start"])] + body * loop["times"] + [(i, False) for i in range(loop["stop"], n)]


def layer(x, i, cfg, W, positions, act=exactly):
    lp, lay, eps = f"l{i}.", cfg["layers"][i], cfg["norm"]["eps"]
    h = act(tanh_norm(x, W, lp + "norm1"))
    if lay["type"] == "retention":
        y = retention(h, positions, W, lp + "mix.", lay["mixer"], eps, act=act)[0]
    else:
        y = latent_attention(h, positions, W, lp + "mix.", lay["mixer"], eps, act)
    x = x + tanh_norm(y, W, lp + "norm1b")
    if lay.get("mlp") is not None:
        x = x + tanh_norm(squared_relu_mlp(act(tanh_norm(x, W, lp + "norm2")), W, lp + "mlp.", act), W, lp + "norm2b")
    return x


def forward(cfg, W, tokens, return_layers=False, act=exactly):
    """Logits [T, vocab] of one sequence from its first token (float64); optionally the stream after every layer run."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    positions = np.arange(len(tokens))
    x0 = embedded(tokens, cfg, W)
    x, after = x0, []
    for i, starts_pass in runs(cfg):
        if starts_pass:
            x = injected(x, x0, W, act)
        x = layer(x, i, cfg, W, positions, act)
        after.append(x)
    logits = softcap(act(tanh_norm(x, W, "final.norm")) @ W["head"].T, cfg.get("logit_softcap"))
    return (logits, np.stack(after)) if return_layers else logits


def bf16_values(a):
    """Rounds to the nearest bfloat16 value (ties to even), kept as float64: a bfloat16 file then holds the weights exactly."""
    f = np.ascontiguousarray(np.asarray(a, dtype=np.float32))
    u = f.view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32)
    return u.view(np.float32).astype(np.float64).reshape(np.shape(a))


def random_weights(cfg, seed=0):
    """Weights for `cfg` (name -> float64 array of bfloat16 values)."""
    rng = np.random.default_rng(seed)
    d, out = int(cfg["width"]), {}

    def put(name, shape, std=None, mean=0.0):
        std = std if std is not None else (1.0 / math.sqrt(shape[-1]) if len(shape) > 1 else 0.5)
        out[name] = bf16_values(rng.standard_normal(shape) * std + mean)

    def norm(name, alpha=0.6):
        put(name, (d,), 0.1, 1.0)
        put(name + ".b", (d,), 0.1)
        put(name + ".alpha", (), 0.05, alpha)

    put("embed", (int(cfg["vocab"]), d), 1.0 / max(1.0, float(cfg["embedding"]["scale"])))
    if cfg["embedding"].get("bigram"):
        put("bigram", (int(cfg["embedding"]["bigram"]["buckets"]) + 1, d), 0.7)
    norm("embed.norm"); norm("final.norm", 0.4)
    put("head", (int(cfg["vocab"]), d))
    if cfg.get("loop"):
        put("loop.in", (d, 2 * d))
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        norm(p + "norm1"); norm(p + "norm1b", 0.9)
        if lay.get("mlp") is not None:
            norm(p + "norm2"); norm(p + "norm2b", 0.9)
            put(p + "mlp.up", (int(lay["mlp"]["ff"]), d), 2.0 / math.sqrt(d))
            put(p + "mlp.down", (d, int(lay["mlp"]["ff"])))
        x = p + "mix."
        H, n, mv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        if lay["type"] == "retention":
            put(x + "q", (H * n, d)); put(x + "k", (H * n, d)); put(x + "v", (H * mv, d)); put(x + "g", (H * mv, d), 2.0 / math.sqrt(d))
            put(x + "o", (d, H * mv), 2.0 / math.sqrt(H * mv))
        else:
            r, rank = int(m["rot_dim"]), int(m["kv_rank"])
            put(x + "q", (H * (n + r), d), 2.0 / math.sqrt(d)); put(x + "dkv", (rank + r, d)); put(x + "dkv.norm", (rank,), 0.1, 1.0)
            put(x + "uk", (H * n, rank)); put(x + "uv", (H * mv, rank)); put(x + "sink", (H,), 1.0)
            put(x + "g", (H, d), 2.0 / math.sqrt(d)); put(x + "o", (d, H * mv), 2.0 / math.sqrt(H * mv))
    return out
