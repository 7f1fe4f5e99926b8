"""The Sofopel decoder through the engine, against the plain implementation (`plain_sofopel.py`).

Every test makes its own small configuration and random weights.  The configurations differ from each other in every size and
constant and exercise the values that are easily 1 or equal: one head and many, keys and values of different widths, groups of one
and of several heads, all of a map rotated, a part and none, windows and chunks of one position, of a page, of a page and one and
longer than the prompt, kept first positions from none to more than a page, convolutions of one to six taps and none, loops that
start at the first layer, later, and none, layers without feed-forward, sizes that are multiples of 8 (the tensor-core kernels)
and sizes that are not (the plain ones).  Where random weights would hide a fault the inputs are made: one key whose score stands
out, placed just inside and just outside a window's or a chunk's edge.
"""
import numpy as np
import pytest
import torch

import ghost_infer_b200 as gi
import plain_sofopel as ps

pytestmark = pytest.mark.gpu


def dif(heads, kv, dim, vdim, chunk, scale, diff=0.3, conv=4, rot=None, base=10000.0):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if conv:
        m["conv"] = conv
    if chunk:
        m["mask"] = {"size": chunk}
    return dict(m, rot={"base": base, "dims": rot}) if rot else m


def win(heads, kv, dim, vdim, window, scale, keep=0, rot=None, base=10000.0, yarn=(2.0, 40.0, 8.0, 1.0)):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if yarn:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return m


def gla(heads, dim, vdim, tau):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def layer(kind, m, ff=None, limit=2.0):
    return {"type": {"D": "attention", "W": "attention_2", "G": "gla"}[kind], "mixer": m, "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def model_cfg(width, vocab, layers, loop=None, scale=1.0, mult=1.0, eps=1e-5):
    cfg = {"architecture": "Sofopel", "width": width, "vocab": vocab, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers,
           "residual_mult": mult}
    return dict(cfg, loop=dict(zip(("start", "stop", "times"), loop))) if loop is not None else cfg


# multiples of 8 throughout; a loop in the middle
CFG_A = model_cfg(64, 150, [
    layer("G", gla(2, 16, 24, 4.0), 48, 1.2),
    layer("D", dif(4, 2, 16, 24, 33, 0.3, 0.15, rot=8, base=900.0), 40),
    layer("W", win(6, 2, 24, 16, 40, 0.25, 3, rot=24, base=5000.0), 64, 0.7),
    layer("G", gla(3, 32, 8, 1.0)),
    layer("W", win(8, 8, 16, 32, 64, 0.3, 70, rot=8, base=100.0), 24),
], loop=(1, 3, 3), scale=3.0, mult=0.4)
# nothing a multiple of 8, the width not even of 4; the loop starts at the first layer and runs to the last; one head
CFG_B = model_cfg(54, 301, [
    layer("D", dif(3, 1, 6, 5, 1, 0.45, 0.8, conv=2, rot=2, base=77.0), 9),
    layer("G", gla(1, 5, 7, 16.0)),
    layer("W", win(1, 1, 10, 6, 65, 0.3, 1, rot=4, base=30.0, yarn=(5.0, 9.0, 3.0, 0.2)), 31, 3.0),
    layer("D", dif(2, 2, 7, 9, 65, 0.3, 0.05, conv=6, rot=6), 14),
    layer("G", gla(5, 6, 3, 0.5), 7),
    layer("W", win(4, 2, 6, 11, 1, 0.6, 0)),
], loop=(0, 6, 2), mult=0.45, eps=3e-6)
# heads as wide as a served model's (the tcgen05 attention takes them), keys wider than any tensor-core kernel takes
CFG_C = model_cfg(128, 150, [
    layer("D", dif(2, 1, 64, 128, 100, 0.1, rot=64, base=1e6), 128),
    layer("G", gla(2, 128, 64, 8.0), 96),
    layer("W", win(4, 1, 128, 128, 70, 0.08, 5, rot=128, base=250000.0), 128),
    layer("D", dif(1, 1, 72, 40, None, 0.1, conv=None)),
    layer("G", gla(1, 200, 40, 16.0)),
    layer("W", win(12, 1, 64, 64, 128, 0.12, 64, rot=32, yarn=None), 64),
], loop=(2, 3, 1), scale=0.5, mult=1.0)
# no loop at all; masks longer than any prompt or absent; one tap
CFG_D = model_cfg(40, 90, [
    layer("W", win(2, 1, 8, 16, 500, 0.3, 2, rot=8), 24),
    layer("D", dif(2, 2, 8, 8, 500, 0.3, conv=1, rot=4), 24),
    layer("G", gla(2, 8, 8, 3.0), 24),
    layer("W", win(6, 3, 8, 8, None, 0.3)),
], mult=0.25)
CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}
RANKS = {"A": 16, "B": {1: 3, 4: 1}, "C": {1: 24, 4: 70}, "D": 8}
_made = {}


def tensors_of(w, bf16=True):
    out = {k: torch.from_numpy(np.array(v, dtype=np.float32)) for k, v in w.items()}
    return {k: v.to(torch.bfloat16) for k, v in out.items()} if bf16 else out


def made(name):
    if name not in _made:
        cfg = CONFIGS[name]
        w = ps.random_weights(cfg, seed=ord(name), rank=RANKS[name])
        _made[name] = (cfg, w, tensors_of(w))
    return _made[name]


def engine_of(cfg, tensors, dtype, max_tokens=64 * 40, max_slots=None, max_seq_len=4096):
    model = gi.Model.from_config_dict(cfg).bind(tensors, dtype, "cuda:0")
    cache = model.new_cache(max_tokens=max_tokens, max_seq_len=max_seq_len, max_slots=max_slots, beyond_trained_positions=True)
    return gi.Engine(model, cache)


def engine_for(name, dtype, **kw):
    cfg, _, tensors = made(name)
    return engine_of(cfg, tensors, dtype, **kw)


_plain = {}


class Reference:
    """The plain logits of a sequence, and per position how far 16-bit roundings may move them: the largest of a few runs of the
    plain implementation with its intermediate numbers shaken (a head whose read-out or whose difference of maps nearly vanishes
    is normed all the same, so some positions feel a rounding far more than others)."""

    def __init__(self, cfg, w, tokens):
        self.cfg, self.w, self.tokens = cfg, w, list(tokens)
        self.logits = ps.forward(cfg, w, self.tokens)
        self._spread = None

    @property
    def spread(self):
        if self._spread is None:
            runs_ = [ps.forward(self.cfg, self.w, self.tokens, act=ps.shaken(s)) - self.logits for s in range(6)]
            self._spread = np.max([np.sqrt((r ** 2).mean(axis=1)) for r in runs_], axis=0)
        return self._spread

    def at(self, rows):
        return Rows(self, rows)


class Rows:
    """Some positions of a `Reference`."""

    def __init__(self, whole, rows):
        self.whole, self.rows, self.logits = whole, rows, whole.logits[rows]

    @property
    def spread(self):
        return self.whole.spread[self.rows]


def plain(name, tokens):
    key = (name, tuple(tokens))
    if key not in _plain:
        cfg, w, _ = made(name)
        _plain[key] = Reference(cfg, w, tokens)
    return _plain[key]


def toks(name, n, seed):
    return np.random.default_rng(seed).integers(0, CONFIGS[name]["vocab"], size=n).tolist()


def check(got, ref, dtype, what=""):
    """32-bit: sums of a few hundred terms over a few dozen dependent stages, relative to the largest logit; at a position that
    feels roundings more than that, a 2,048th of what shaking the plain implementation's intermediate numbers (by roundings 65,536
    times as large) does there.  bfloat16: per
    position, four times what shaking the plain implementation's intermediate numbers does there (never less than it does
    to the middle position), with room for one position in 25 whose read-out nearly vanished in a way no shaking met; most
    positions must be ones that feel little.  A key one position off, a lost state, a wrong tap or
    a wrong angle moves logits by tens of percent of their spread."""
    got = np.asarray(got, dtype=np.float64)
    assert got.shape == ref.logits.shape, f"{what}: {got.shape} vs {ref.logits.shape}"
    assert np.isfinite(got).all(), f"{what}: non-finite logits"
    scale = max(1.0, float(np.abs(ref.logits).max()))
    err = np.abs(got - ref.logits)
    if dtype == "float32":
        if err.max() <= 5e-5 * scale:
            return
        limit = np.maximum(5e-5 * scale, ref.spread / 2048.0)
        assert (err.max(axis=1) <= 4.0 * limit).all() and (np.sqrt((err ** 2).mean(axis=1)) <= limit).all(), f"{what}: max error {err.max():.3e} (scale {scale:.2f}) at {np.unravel_index(err.argmax(), err.shape)}"
        return
    rms = np.sqrt((err ** 2).mean(axis=1))
    limit = 4.0 * np.maximum(ref.spread, np.median(ref.spread))
    ratio = rms / limit
    assert (ratio > 1.0).sum() <= max(1, len(rms) // 25) and ratio.max() <= 4.0, \
        f"{what}: {(ratio > 1.0).sum()} of {len(rms)} positions are off, position {int(ratio.argmax())} by {ratio.max():.2f} of its limit {limit[ratio.argmax()]:.3e}"
    assert len(rms) < 20 or np.median(limit) <= 0.25 * np.sqrt((ref.logits ** 2).mean()), f"{what}: the limits are too wide to tell a fault ({np.median(limit):.3e})"


def run_whole(eng, tokens):
    s = eng.cache.open_slot()
    out = eng.step([gi.StepEntry(s, tokens, list(range(len(tokens))))]).cpu().numpy()
    eng.cache.close_slot(s)
    return out


def prompt_then_tokens(eng, t, cut, graph=None):
    """The first `cut` tokens in one step, the rest one by one through the decode runner."""
    s = eng.cache.open_slot()
    rows = [eng.step([gi.StepEntry(s, t[:cut], list(range(cut)))]).cpu().numpy()]
    run = eng.decoder([s]) if graph is None else eng.decoder([s], use_graph=graph)
    rows += [run.forward(tokens=[x]).cpu().numpy().copy() for x in t[cut:]]
    eng.cache.close_slot(s)
    return np.concatenate(rows, 0)


PATHS = [(n, d) for d in ("float32", "bfloat16") for n in sorted(CONFIGS)]


# ---- kernels by themselves, against 64-bit torch ----------------------------------------------------------------------------
@pytest.mark.parametrize("rows,width", [(5, 52), (3, 54), (70, 1028), (300, 7), (9, 1), (700, 512), (2, 4096), (3, 8192), (1, 20000), (600, 4096)])
def test_the_pass_that_joins_a_layer_to_the_stream(rows, width):
    from ghost_infer_b200.kernels import ops
    from ghost_infer_b200.parts import RowRead
    g = torch.Generator(device="cuda:0").manual_seed(rows * 1000 + width)
    rnd = lambda *shape: torch.randn(shape, device="cuda:0", generator=g)
    x, y, w = rnd(rows, width), rnd(rows, width), rnd(width)
    want = x.double() + 0.3 * y.double()
    normed = want / torch.sqrt((want ** 2).mean(-1, keepdim=True) + 1e-5) * w.double()
    x1, y1 = x.clone(), y.clone()
    h = ops.join_rows(x1, y1, 0.3, RowRead(w, 1e-5, torch.float32))
    torch.testing.assert_close(x1.double(), want, rtol=1e-6, atol=1e-6)
    torch.testing.assert_close(h.double(), normed, rtol=1e-5, atol=1e-5)
    assert float(y1.abs().max()) == 0.0
    x2, y2 = x.clone(), y.clone()
    h16 = ops.join_rows(x2, y2, 0.3, RowRead(w.bfloat16(), 1e-5, torch.bfloat16))
    want16 = want / torch.sqrt((want ** 2).mean(-1, keepdim=True) + 1e-5) * w.bfloat16().double()
    torch.testing.assert_close(h16.double(), want16, rtol=5e-3, atol=1e-5)
    x3, y3 = x.clone(), y.clone()
    assert ops.join_rows(x3, y3, 0.3) is None
    assert torch.equal(x3, x1) and float(y3.abs().max()) == 0.0


@pytest.mark.parametrize("m,width", [(1, 4096), (7, 2048), (16, 256), (3, 6144)])
@pytest.mark.parametrize("normed", [True, False])
def test_joining_rows_with_partial_sums(m, width, normed):
    from ghost_infer_b200.kernels import ops
    from ghost_infer_b200.parts import RowRead
    g = torch.Generator(device="cuda:0").manual_seed(m + width)
    k = 1024
    a = torch.randn((m, k), device="cuda:0", generator=g).bfloat16()
    w = (torch.randn((width, k), device="cuda:0", generator=g) / k ** 0.5).bfloat16()
    x, nw = torch.randn((m, width), device="cuda:0", generator=g), torch.rand((width,), device="cuda:0", generator=g) + 0.5
    y = ops.as_carrier(torch.randn((m, width), device="cuda:0", generator=g))
    want = x.double() + 0.7 * (y.as_subclass(torch.Tensor).double() + a.double() @ w.double().T)
    with ops.defer_into(y):
        ops.linear(a, w, out=y, accumulate=True)
    x1 = ops.as_carrier(x.clone())
    h = ops.join_rows(x1, y, 0.7, RowRead(nw, 1e-5, torch.float32) if normed else None)
    torch.testing.assert_close(x1.as_subclass(torch.Tensor).double(), want, rtol=1e-5, atol=2e-5)
    assert not ops.has_pending(y) and float(y.as_subclass(torch.Tensor).abs().max()) == 0.0
    if normed:
        torch.testing.assert_close(h.double(), want / torch.sqrt((want ** 2).mean(-1, keepdim=True) + 1e-5) * nw.double(), rtol=2e-5, atol=2e-5)


@pytest.mark.parametrize("m,width", [(1, 4096), (16, 2048), (3, 1536), (8, 8192)])
def test_partial_sums_of_two_products(m, width):
    """Two products into the same rows leave their cut tiles pending side by side: the join adds both, as does anyone else who reads
    the rows; a product stored for another reader in between does not disturb them."""
    from ghost_infer_b200.kernels import ops
    g = torch.Generator(device="cuda:0").manual_seed(m + width)
    rnd = lambda *s: torch.randn(s, device="cuda:0", generator=g)
    k1, k2 = 1024, 1536
    a1, a2 = rnd(m, k1).bfloat16(), rnd(m, k2).bfloat16()
    w1, w2 = (rnd(width, k1) / k1 ** 0.5).bfloat16(), (rnd(width, k2) / k2 ** 0.5).bfloat16()
    x, y0 = rnd(m, width), rnd(m, width)
    total = y0.double() + a1.double() @ w1.double().T + a2.double() @ w2.double().T
    for how in ("join", "settle", "torch", "third", "norm"):
        y = ops.as_carrier(y0.clone())
        with ops.defer_into(y, two=True):
            ops.linear(a1, w1, out=y, accumulate=True)
            with ops.defer_store():
                ops.linear(a2, w2, out_dtype=torch.bfloat16)
            ops.linear(a2, w2, out=y, accumulate=True)
            if how == "third":
                ops.linear(a1, w1, out=y, accumulate=True)
        if how == "join":
            x1 = ops.as_carrier(x.clone())
            ops.join_rows(x1, y, 0.7)
            torch.testing.assert_close(x1.as_subclass(torch.Tensor).double(), x.double() + 0.7 * total, rtol=1e-5, atol=3e-5)
            assert float(y.as_subclass(torch.Tensor).abs().max()) == 0.0
        elif how == "norm":
            h = ops.rmsnorm(y, torch.ones((width,), device="cuda:0"), 1e-5, torch.float32)
            torch.testing.assert_close(h.double(), total / torch.sqrt((total ** 2).mean(-1, keepdim=True) + 1e-5), rtol=2e-5, atol=2e-5)
        else:
            got = (y + 0.0) if how == "torch" else y
            if how != "torch":
                ops.settle(y)
            want = total + (a1.double() @ w1.double().T if how == "third" else 0.0)
            torch.testing.assert_close(got.as_subclass(torch.Tensor).double(), want, rtol=1e-5, atol=3e-5)
        assert not ops.has_pending(y) and "_gi_pending2" not in y.__dict__


@pytest.mark.parametrize("heads,kv,dim,vdim,taps,rot,adjacent", [(4, 2, 16, 24, 4, 8, True), (2, 1, 64, 128, 4, 64, True), (3, 3, 8, 12, 3, 6, True),
                                                                 (3, 1, 6, 5, 2, 2, True), (2, 2, 7, 9, 6, 6, True), (4, 2, 12, 8, 2, 12, False),
                                                                 (1, 1, 4, 4, 1, 0, True), (5, 5, 8, 4, 0, 4, True)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_maps_prepared_across_portions_and_in_a_batch(heads, kv, dim, vdim, taps, rot, adjacent, dtype):
    """Three sequences fed in portions of unequal sizes down to one token, with padding rows between: convolution (inputs of
    earlier portions from the state), rotation, the two maps' places in queries and cache."""
    from ghost_infer_b200.cache.sequence_cache import CacheRequest, SequenceCache, StateRequest
    from ghost_infer_b200.kernels import ops
    dt = getattr(torch, dtype)
    channels = 2 * dim * (heads + kv) + kv * vdim
    rng = np.random.default_rng(channels)
    lens = [70, 9, 133]
    rows = [rng.standard_normal((n, channels)).astype(np.float32) for n in lens]
    cw = rng.standard_normal((channels, taps)).astype(np.float32) if taps else None
    cache = SequenceCache([(0, CacheRequest("full", kv, 2 * dim, None, vdim), StateRequest(((taps - 1) * channels,)) if taps > 1 else None, None)],
                          max_tokens=64 * 8, max_slots=4, max_seq_len=256, dtype=dt, device="cuda:0")
    slots = [cache.open_slot() for _ in lens]
    cuts = [[0, 2, 3, 4, 40, 66, 70], [0, 1, 1, 5, 6, 8, 9], [0, 64, 65, 66, 67, 129, 133]]
    conv = torch.from_numpy(np.ascontiguousarray(cw.T)).cuda() if taps else None
    got = [[] for _ in lens]
    freq = 100.0 ** (-2.0 * np.arange(rot // 2) / max(rot, 1))
    for k in range(6):
        part = [(i, cuts[i][k], cuts[i][k + 1]) for i in (2, 0, 1) if cuts[i][k + 1] > cuts[i][k]]
        cache.reserve([(slots[i], b) for i, a, b in part])
        cache.sync_tables()
        one = all(b - a == 1 for _, a, b in part)
        pos = np.concatenate([np.arange(a, b) for _, a, b in part] + ([[0, 0]] if one else []))
        sl = np.concatenate([np.full(b - a, slots[i]) for i, a, b in part] + ([[-1, -1]] if one else []))
        flat = np.concatenate([rows[i][a:b] for i, a, b in part] + ([np.zeros((2, channels), np.float32)] if one else []))
        cu = np.concatenate([[0], np.cumsum([b - a for _, a, b in part])])
        i32 = lambda v: torch.tensor(np.asarray(v), dtype=torch.int32, device="cuda:0")
        step = type("S", (), {})()
        step.positions, step.token_slots, step.cu_seqlens = i32(pos), i32(sl), i32(cu)
        step.seq_slots, step.n_seqs, step.is_decode = i32([slots[i] for i, _, _ in part]), len(part), one
        ang = pos[:, None] * freq[None, :]
        table = torch.from_numpy(np.stack([np.cos(ang), np.sin(ang)], -1).astype(np.float32)).cuda() if rot else None
        mem = cache.memory(0)
        q = ops.map_prepare(torch.from_numpy(flat).cuda(), dt, conv, mem.state, table, rot, adjacent, step, mem, heads, kv, dim, vdim)
        at = 0
        for i, a, b in part:
            got[i].append(q[at:at + b - a].double().cpu().numpy())
            at += b - a
            cache.commit(slots[i], b)
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == "float32" else dict(rtol=1e-2, atol=1e-2)
    for i, n in enumerate(lens):
        u = ps.short_conv(rows[i].astype(np.float64), cw.astype(np.float64)) if taps else rows[i].astype(np.float64)
        spec = {"dims": rot, "base": 100.0}
        qd, kd = heads * 2 * dim, kv * 2 * dim
        wq = ps.rotate(u[:, :qd].reshape(n, heads, 2, dim), np.arange(n), spec, "adjacent" if adjacent else "half")
        wk = ps.rotate(u[:, qd:qd + kd].reshape(n, kv, 2, dim), np.arange(n), spec, "adjacent" if adjacent else "half")
        full = np.zeros((n, heads, 2, 2, dim))
        full[:, :, 0, 0], full[:, :, 1, 1] = wq[:, :, 0], wq[:, :, 1]
        assert np.allclose(np.concatenate(got[i]), full.reshape(n, -1), **tol), f"queries of sequence {i}"
        bt = cache.memory(0).block_table[slots[i]].cpu().numpy()
        k, v = cache.memory(0).k.double().cpu().numpy(), cache.memory(0).v.double().cpu().numpy()
        for p in range(n):
            assert np.allclose(k[bt[p // 64], :, p % 64], wk[p].reshape(kv, 2 * dim), **tol), f"key {p} of sequence {i}"
            assert np.allclose(v[bt[p // 64], :, p % 64], u[p, qd + kd:].reshape(kv, vdim), **tol), f"value {p} of sequence {i}"


@pytest.mark.parametrize("rows,heads,width", [(3, 4, 64), (70, 3, 128), (5, 2, 300), (9, 5, 7), (2, 1, 600), (1, 2, 512)])
def test_difference_of_maps(rows, heads, width):
    from ghost_infer_b200.kernels import ops
    a = torch.randn((rows, heads * 2 * width), device="cuda:0", generator=torch.Generator(device="cuda:0").manual_seed(rows + width))
    u = a.double().view(rows, heads, 2, width).cpu().numpy()
    want = ps.difference_of_maps(u[:, :, 0], u[:, :, 1], 0.45, 0.3, 1e-5).reshape(rows, -1)
    got = ops.map_difference(a, heads, width, 0.45, 0.7, 1e-5)
    assert np.allclose(got.double().cpu().numpy(), want, rtol=1e-5, atol=1e-5)
    b = a.bfloat16()
    u = b.double().view(rows, heads, 2, width).cpu().numpy()
    want = ps.difference_of_maps(u[:, :, 0], u[:, :, 1], 0.45, 0.3, 1e-5).reshape(rows, -1)
    assert np.allclose(ops.map_difference(b, heads, width, 0.45, 0.7, 1e-5).double().cpu().numpy(), want, rtol=5e-3, atol=1e-4)


@pytest.mark.parametrize("rows,rank,channels,tau", [(5, 16, 96, 16.0), (70, 3, 300, 1.0), (1, 1, 7, 0.25), (9, 130, 64, 5.0)])
def test_decays_per_key(rows, rank, channels, tau):
    from ghost_infer_b200.kernels import ops
    g = torch.Generator(device="cuda:0").manual_seed(rank)
    rnd = lambda *s: torch.randn(s, device="cuda:0", generator=g)
    wide, up, b = rnd(rows, rank + 8), rnd(rank, channels) / rank ** 0.5, 4.0 * rnd(channels)
    b[0], b[-1] = 60.0, -60.0                     # a channel that keeps everything, one that keeps nothing
    low = wide[:, 3:3 + rank]
    for x in (low, wide.bfloat16()[:, 3:3 + rank]):
        z = x.double() @ up.double() + b.double()
        want = torch.exp(-torch.nn.functional.softplus(-z, threshold=1e9) / tau)
        torch.testing.assert_close(ops.key_decays(x, up, b, tau).double(), want, rtol=2e-5, atol=1e-30)


@pytest.mark.parametrize("K,V,heads", [(16, 24, 2), (40, 56, 3), (5, 7, 1), (64, 130, 2), (128, 64, 2), (200, 40, 1), (256, 8, 1), (6, 3, 5), (30, 33, 2)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_recurrence_with_decays_per_key(K, V, heads, dtype):
    """Sequences in portions, among others one token each (the other instance of the kernel), with decays from 0 to 1; the state
    goes on from what earlier portions left.  32-bit: the same bits however the tokens are cut."""
    from ghost_infer_b200.kernels import ops
    dt = getattr(torch, dtype)
    g = torch.Generator(device="cuda:0").manual_seed(K * V)
    lens = [77, 5, 40]
    rnd = lambda *s: torch.randn(s, device="cuda:0", generator=g)
    seqs = []
    for n in lens:
        a = torch.rand((n, heads * K), device="cuda:0", generator=g) ** 0.2
        a[:, 0] = 1.0
        a[::3, -1] = 0.0
        seqs.append((rnd(n, heads * K).to(dt), (rnd(n, heads * K) / K ** 0.5).to(dt), rnd(n, heads * V).to(dt), a))
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda:0")

    def run(cuts):
        state = torch.zeros((5, heads * K * V + 4), dtype=torch.float32, device="cuda:0")
        outs = [[] for _ in lens]
        for k in range(len(cuts[0]) - 1):
            part = [(i, cuts[i][k], cuts[i][k + 1]) for i in (1, 0, 2) if cuts[i][k + 1] > cuts[i][k]]
            cat = [torch.cat([seqs[i][j][a:b] for i, a, b in part]).contiguous() for j in range(4)]
            step = type("S", (), {})()
            step.cu_seqlens = i32(np.concatenate([[0], np.cumsum([b - a for _, a, b in part])]).tolist())
            step.seq_slots, step.n_seqs = i32([i + 1 for i, _, _ in part]), len(part)
            o = ops.linear_state_keyed(*cat, state, step, heads, K, V, 0.37)
            at = 0
            for i, a, b in part:
                outs[i].append(o[at:at + b - a])
                at += b - a
        return [torch.cat(o) for o in outs]

    whole = run([[0, n] for n in lens])
    cut = run([[0, 2, 20, 21, 77], [0, 1, 3, 4, 5], [0, 0, 33, 34, 40]])
    for i, n in enumerate(lens):
        assert torch.equal(whole[i], cut[i]), f"sequence {i} depends on the cut"
        q, k, v, a = (t.double().cpu().numpy().reshape(n, heads, -1) for t in seqs[i])
        S, want = np.zeros((heads, K, V)), np.zeros((n, heads, V))
        for t in range(n):
            S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
            want[t] = 0.37 * np.einsum("hnm,hn->hm", S, q[t])
        err = np.abs(whole[i].double().cpu().numpy() - want.reshape(n, -1)).max()
        assert err <= 3e-5 * max(1.0, np.abs(want).max()), f"sequence {i}: {err:.2e}"


@pytest.mark.parametrize("rows", [1, 5, 64, 65, 300])
@pytest.mark.parametrize("ff,width", [(48, 64), (320, 256), (7, 54), (2048, 512)])
def test_clamped_feed_forward_part(rows, ff, width):
    from ghost_infer_b200.parts import Runtime, lookup
    g = torch.Generator(device="cuda:0").manual_seed(rows + ff)
    rnd = lambda *s: torch.randn(s, device="cuda:0", generator=g)
    h, w = rnd(rows, width), {"gate": 2 * rnd(ff, width) / width ** 0.5, "up": 2 * rnd(ff, width) / width ** 0.5, "down": rnd(width, ff) / ff ** 0.5}
    part = lookup("feed_forward", "gated_mlp")({"hidden_size": width, "intermediate_size": ff, "activation": "clamped", "limit": 1.3, "alpha": 1.702,
                                                "tensor_names": {k: k for k in w}}, "")
    for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
        ws = {k: v.to(dt) for k, v in w.items()}
        part.bind(ws, Runtime(torch.device("cuda:0"), dt))
        a = h.to(dt)
        out = torch.zeros((rows, width), dtype=torch.float32, device="cuda:0")
        part.forward(a, out, None)
        want = ps.clamped_gated_mlp(a.double().cpu().numpy(), {k: v.double().cpu().numpy() for k, v in ws.items()}, "", 1.3)
        assert np.abs(out.double().cpu().numpy() - want).max() <= tol * max(1.0, np.abs(want).max())


# ---- the arrangement by itself ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("what", ["both", "mixer", "feed-forward"])
@pytest.mark.parametrize("reader", [True, False])
def test_parallel_block(what, reader):
    from ghost_infer_b200.kernels import ops
    from ghost_infer_b200.parts import FeedForward, Mixer, Runtime, lookup
    d, T = 48, 9
    g = torch.Generator(device="cuda:0").manual_seed(2)
    ws = {f"n{i}": torch.rand((d,), device="cuda:0", generator=g) + 0.5 for i in range(2)}
    norms = [lookup("norm", "rmsnorm")({"size": d, "eps": 1e-5, "tensor_names": {"weight": ""}}, n) for n in ws]
    for n in norms:
        n.bind(ws, Runtime(torch.device("cuda:0"), torch.float32))
    a, b = (torch.randn((d, d), device="cuda:0", generator=g) / d ** 0.5 for _ in range(2))

    class Mix(Mixer):
        def forward(self, h, residual, step, memory):
            residual += h @ a.T

    class Ffn(FeedForward):
        def forward(self, h, residual, step):
            residual += h @ b.T

    block = lookup("block", "parallel_residual")(norms[0], Mix({}) if what != "feed-forward" else None, None, Ffn({}) if what != "mixer" else None)
    block.params = {"scale": -0.35}
    step = type("S", (), {"shared": {}, "next_reader": norms[1] if reader else None})()
    x = ops.as_carrier(torch.randn((T, d), device="cuda:0", generator=g))
    rms = lambda u, w: u / torch.sqrt((u ** 2).mean(-1, keepdim=True) + 1e-5) * w.double()
    want = x.as_subclass(torch.Tensor).double()
    for _ in range(2):                                     # twice: the rows the sublayers add into are zero again
        h = rms(want, ws["n0"])
        want = want - 0.35 * ((h @ a.double().T if what != "feed-forward" else 0) + (h @ b.double().T if what != "mixer" else 0))
        block.forward(x, step, None)
    torch.testing.assert_close(x.as_subclass(torch.Tensor).double(), want, rtol=1e-5, atol=1e-5)
    left = x.__dict__.get("_gi_handed")
    assert (left is not None) == reader
    torch.testing.assert_close(norms[1].forward(x).double(), rms(want, ws["n1"]), rtol=1e-5, atol=1e-5)


# ---- each mechanism alone: one- and two-layer models ------------------------------------------------------------------------
ALONE = {
    "maps": ([layer("D", dif(3, 1, 6, 5, 7, 0.4, conv=None))], {}),
    "maps_one_head": ([layer("D", dif(1, 1, 4, 4, None, 0.5, 0.0, conv=None))], {}),
    "maps_turned": ([layer("D", dif(4, 2, 8, 12, 100, 0.3, conv=None, rot=8, base=50.0))], {}),
    "maps_turned_in_part": ([layer("D", dif(2, 2, 10, 8, 33, 0.3, conv=None, rot=4))], {}),
    "convolution": ([layer("D", dif(2, 1, 8, 8, 16, 0.3, conv=4))], {}),
    "convolution_of_one_tap": ([layer("D", dif(2, 1, 8, 8, 16, 0.3, conv=1))], {}),
    "convolution_of_seven_taps": ([layer("D", dif(2, 2, 4, 8, 16, 0.3, conv=7, rot=2))], {}),
    "chunk_of_one": ([layer("D", dif(2, 1, 8, 8, 1, 0.3, conv=3))], {}),
    "window": ([layer("W", win(4, 2, 6, 9, 7, 0.4))], {}),
    "window_of_one_and_the_first": ([layer("W", win(2, 1, 8, 8, 1, 0.4, 1, rot=8))], {}),
    "window_and_many_first": ([layer("W", win(2, 2, 8, 8, 5, 0.4, 20, rot=4, yarn=None))], {}),
    "window_yarn": ([layer("W", win(3, 3, 16, 4, 64, 0.4, 2, rot=16, base=500.0, yarn=(8.0, 16.0, 4.0, 0.5)))], {}),
    "window_longer_than_the_prompt": ([layer("W", win(2, 1, 8, 8, 500, 0.4, 3))], {}),
    "decay_per_key": ([layer("G", gla(3, 6, 9, 4.0))], {}),
    "decay_one_head_no_root": ([layer("G", gla(1, 4, 4, 1.0))], {}),
    "decay_widest_keys": ([layer("G", gla(1, 256, 4, 16.0))], {}),
    "feed_forward": ([layer("G", gla(1, 4, 4, 2.0), 30, 0.4)], {}),
    "scaled": ([layer("G", gla(2, 4, 8, 2.0), 12), layer("W", win(2, 1, 8, 8, 9, 0.4), 8)], {"scale": 5.0, "mult": 0.15}),
    "loop_over_everything": ([layer("G", gla(2, 4, 4, 8.0), 8), layer("D", dif(2, 1, 4, 4, 9, 0.4), 8)], {"loop": (0, 2, 3), "mult": 0.5}),
    "loop_of_one_layer_at_the_end": ([layer("W", win(2, 1, 4, 4, 9, 0.4), 8), layer("D", dif(2, 2, 4, 4, 9, 0.4))], {"loop": (1, 2, 4), "mult": 0.5}),
    "loop_of_one_pass": ([layer("G", gla(2, 4, 4, 8.0), 8)], {"loop": (0, 1, 1)}),
}


@pytest.mark.parametrize("which", sorted(ALONE))
@pytest.mark.parametrize("width", [48, 45])
def test_each_mechanism_alone(which, width):
    layers, opts = ALONE[which]
    cfg = model_cfg(width, 90, layers, **opts)
    w = ps.random_weights(cfg, seed=11)
    eng = engine_of(cfg, tensors_of(w, False), "float32", max_tokens=256, max_seq_len=256)
    t = np.random.default_rng(5).integers(0, 90, size=70).tolist()
    ref = Reference(cfg, w, t)
    check(run_whole(eng, t), ref, "float32", which)
    check(prompt_then_tokens(eng, t, 30), ref, "float32", which + ", decoded")


def test_the_stream_after_every_layer_run():
    cfg, w, tensors = made("A")
    eng = engine_of(cfg, tensors, "float32")
    seen = []
    for lay in eng.model.layers:
        def spied(x, step, memory, run=lay.block.forward):
            run(x, step, memory)
            seen.append(x.as_subclass(torch.Tensor).double().cpu().numpy())
        lay.block.forward = spied
    t = toks("A", 50, 3)
    run_whole(eng, t)
    _, after = ps.forward(cfg, w, t, return_layers=True)
    assert len(seen) == len(after) == 9
    for i, (got, ref) in enumerate(zip(seen, after)):
        assert np.abs(got - ref).max() <= 5e-5 * np.abs(ref).max(), f"after run {i}"


# ---- keys far away, and just inside and just outside every edge ------------------------------------------------------------
def standing_out(kind, m, query_at, key_at, width=64, vocab=40, n=None):
    """A one-layer model in which token 1 (at `key_at`) carries the key that token 2's query (at `query_at`) looks for, far above
    all other scores, and token 1's value moves the logits; every other token is 0 and carries almost nothing."""
    cfg = model_cfg(width, vocab, [layer(kind, m)], mult=2.0)
    w = {k: np.array(v) for k, v in ps.random_weights(cfg, seed=9).items()}
    p, rng = "l0.mix.", np.random.default_rng(3)
    basis = np.eye(width)
    w["embed"][:] = 0.05 * rng.standard_normal((vocab, width)); w["embed"][:, :2] = 0.0     # nothing of what tokens 1 and 2 carry
    w["embed"][1] = 8 * basis[0]; w["embed"][2] = 8 * basis[1]
    H, G, nd = m["heads"], m["kv_heads"], m["dim"]
    maps = 2 if kind == "D" else 1
    direction = rng.standard_normal((nd,)); direction[:m["rot"]["dims"] if m.get("rot") else 0] = 0.0       # what does not turn
    direction *= 1.0 / np.sqrt((direction ** 2).sum())
    for name, heads, col in (("q", H, 1), ("k", G, 0)):
        w[p + name] = 0.02 * rng.standard_normal(w[p + name].shape)
        one = np.zeros((heads, maps, nd)); one[:, 0] = 12.0 * direction                                       # the first map alone
        w[p + name][:, col] = one.reshape(-1)
    w[p + "v"] = 0.02 * rng.standard_normal(w[p + "v"].shape)
    w[p + "v"][:, 0] = 2.0 * rng.standard_normal(w[p + "v"].shape[0])
    if kind == "D":
        for name in "qkv":                                                                                    # the token's own tap alone
            w[p + name + ".conv"] = np.zeros_like(w[p + name + ".conv"]); w[p + name + ".conv"][:, -1] = 1.0
    w = {k: ps.bf16_values(v) for k, v in w.items()}
    t = [0] * (n or query_at + 1)
    t[key_at], t[query_at] = 1, 2
    return cfg, w, t


EDGES = []
for size in (1, 20, 64, 65):
    for query in (130, 200):
        lo = query - size + 1
        EDGES += [("W", win(4, 2, 16, 16, size, 0.5, 3, rot=8), query, key) for key in {lo, lo - 1, 2, 3} if key < query]
for size in (20, 64, 65, 200):
    for query in (129, 195, 259):
        lo = query // size * size
        EDGES += [("D", dif(4, 2, 16, 32, size, 0.5, rot=8), query, key) for key in {lo, lo - 1} if 0 <= key < query]
EDGES += [("D", dif(4, 2, 16, 32, None, 0.5, rot=8), 300, key) for key in (0, 63, 64)]
EDGES += [("W", win(4, 2, 16, 16, None, 0.5, rot=8), 300, key) for key in (0, 127, 128)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_that_stands_out_at_every_edge(dtype):
    """In prompts, decoded, and with the query's portion starting just before it; seen exactly where the mask says so."""
    for kind, m, query, key in EDGES:
        cfg, w, t = standing_out(kind, m, query, key)
        ref = ps.forward(cfg, w, t)[query]
        blank = ps.forward(cfg, w, t[:key] + [0] + t[key + 1:])[query]
        mask = m.get("mask")
        sees = (key // mask["size"] == query // mask["size"] if kind == "D" else query - key < mask["size"] or key < mask["keep_first"]) if mask else True
        moved = np.abs(ref - blank).max()
        what = f"{kind} {mask} query {query} key {key}"
        assert (moved > 0.5) == sees, f"{what}: the key moves the logits by {moved:.3f}"
        eng = engine_of(cfg, tensors_of(w), dtype, max_tokens=64 * 8, max_seq_len=512)
        limit = (2e-4 if dtype == "float32" else 0.06) * max(1.0, np.abs(ref).max())
        for cut in (0, query, max(1, query - 2)):
            s = eng.cache.open_slot()
            if cut:
                eng.step([gi.StepEntry(s, t[:cut], [])])
            got = eng.step([gi.StepEntry(s, t[cut:], [query - cut])]).cpu().numpy()[0]
            eng.cache.close_slot(s)
            assert np.abs(got - ref).max() <= limit, f"{what} cut at {cut}: {np.abs(got - ref).max():.4f}"


def test_the_one_in_the_denominator_shows():
    """A query whose only visible key scores far below 0 gives almost nothing: without the one it would give the whole value."""
    cfg, w, t = standing_out("W", win(2, 1, 16, 16, 1, 0.5, 0), 40, 10)
    w["l0.mix.q"][:, 1] = 12.0 * np.tile(np.eye(16)[0], 2); w["l0.mix.k"][:, 1] = -12.0 * np.eye(16)[0]
    w["l0.mix.v"][:, 1] = w["l0.mix.v"][:, 0]
    w = {k: ps.bf16_values(v) for k, v in w.items()}
    ref = ps.forward(cfg, w, t)
    for dtype, tol in (("float32", 2e-4), ("bfloat16", 0.06)):
        eng = engine_of(cfg, tensors_of(w), dtype, max_tokens=256, max_seq_len=256)
        for got in (run_whole(eng, t), prompt_then_tokens(eng, t, 39)):
            assert np.abs(got - ref).max() <= tol * max(1.0, np.abs(ref).max())
    for keep in (0, 1):
        without = ps.softmax(np.array([[-30.0]])) if keep else ps.softmax_plus_one(np.array([[-30.0]]))
        assert (without[0, 0] > 0.5) == bool(keep)


# ---- whole prompts, decoding, portions, batches -----------------------------------------------------------------------------
@pytest.mark.parametrize("name,dtype", PATHS)
def test_whole_prompt(name, dtype):
    eng = engine_for(name, dtype)
    for n, seed in ((1, 1), (2, 2), (64, 3), (65, 4), (200, 5)):
        t = toks(name, n, seed)
        check(run_whole(eng, t), plain(name, t), dtype, f"{name} {n} tokens")


@pytest.mark.parametrize("name,dtype", PATHS)
@pytest.mark.parametrize("graph", [False, True])
def test_prompt_then_token_by_token(name, dtype, graph):
    eng = engine_for(name, dtype)
    t = toks(name, 150, 21)          # decoded across the page borders at 64 and 128 and out of every window and chunk
    check(prompt_then_tokens(eng, t, 60, graph), plain(name, t), dtype)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_decoding_from_the_first_token(name):
    eng = engine_for(name, "float32")
    t = toks(name, 80, 8)
    s = eng.cache.open_slot()
    rows = [eng.step([gi.StepEntry(s, [x], [0])]).cpu().numpy() for x in t]
    eng.cache.close_slot(s)
    check(np.concatenate(rows, 0), plain(name, t), "float32")


@pytest.mark.parametrize("name,dtype", PATHS)
def test_portions_of_several_sizes(name, dtype):
    eng = engine_for(name, dtype)
    t = toks(name, 140, 31)
    for cuts in ((2, 4, 66, 130, 140), (63, 64, 65, 128, 140), (1, 3, 5, 7, 140), (20, 40, 41, 43, 110, 140)):
        s = eng.cache.open_slot()
        rows, a = [], 0
        for b in cuts:
            rows.append(eng.step([gi.StepEntry(s, t[a:b], list(range(b - a)))]).cpu().numpy())
            a = b
        eng.cache.close_slot(s)
        check(np.concatenate(rows, 0), plain(name, t), dtype, f"{name} cut at {cuts}")


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_float32_does_not_depend_on_the_cut_or_the_batch(name):
    eng = engine_for(name, "float32")
    t, other = toks(name, 130, 41), toks(name, 20, 42)
    whole = run_whole(eng, t)
    s = eng.cache.open_slot()
    cut = np.concatenate([eng.step([gi.StepEntry(s, t[a:b], list(range(b - a)))]).cpu().numpy() for a, b in ((0, 7), (7, 9), (9, 71), (71, 130))], 0)
    eng.cache.close_slot(s)
    assert np.array_equal(whole, cut)
    s1, s2 = eng.cache.open_slot(), eng.cache.open_slot()
    both = eng.step([gi.StepEntry(s2, other, [0]), gi.StepEntry(s1, t, list(range(130)))]).cpu().numpy()
    eng.cache.close_slot(s1); eng.cache.close_slot(s2)
    assert np.array_equal(whole, both[1:])


@pytest.mark.parametrize("name,dtype", PATHS)
def test_unequal_batch_against_each_alone(name, dtype):
    eng = engine_for(name, dtype)
    prompts = [toks(name, n, 50 + n) for n in (90, 3, 66, 1, 130)]
    tails = 6
    slots = [eng.cache.open_slot() for _ in prompts]
    cut = [max(1, len(p) - tails) for p in prompts]
    out = eng.step([gi.StepEntry(s, p[:c], list(range(c))) for s, p, c in zip(slots, prompts, cut)]).cpu().numpy()
    got = [[out[sum(cut[:i]):sum(cut[:i + 1])]] for i in range(len(prompts))]
    fed = list(cut)
    while True:
        live = [i for i in range(len(prompts)) if fed[i] < len(prompts[i])]
        if not live:
            break
        run = eng.decoder([slots[i] for i in live])          # the shorter requests end earlier; three rows are padded to four
        rows = run.forward(tokens=[prompts[i][fed[i]] for i in live]).cpu().numpy()
        for k, i in enumerate(live):
            got[i].append(rows[k:k + 1].copy())
            fed[i] += 1
    for s in slots:
        eng.cache.close_slot(s)
    for i, p in enumerate(prompts):
        check(np.concatenate(got[i], 0), plain(name, p), dtype, f"{name}: request {i} of the batch")


def test_mixed_step_of_fresh_prompts_and_sequences_under_way():
    """One step holds the second portion of one request and the whole of another: positions, chunks and taps count from 0 in each."""
    for name in ("A", "B"):
        eng = engine_for(name, "float32")
        a, b = toks(name, 120, 61), toks(name, 40, 62)
        s1, s2 = eng.cache.open_slot(), eng.cache.open_slot()
        r0 = eng.step([gi.StepEntry(s1, a[:50], list(range(50)))]).cpu().numpy()
        r1 = eng.step([gi.StepEntry(s2, b, list(range(40))), gi.StepEntry(s1, a[50:110], list(range(60)))]).cpu().numpy()
        r2 = eng.step([gi.StepEntry(s1, a[110:], list(range(10)))]).cpu().numpy()
        eng.cache.close_slot(s1); eng.cache.close_slot(s2)
        check(np.concatenate([r0, r1[40:], r2], 0), plain(name, a), "float32", "under way")
        check(r1[:40], plain(name, b), "float32", "fresh")


# ---- pages and slots given back and used again --------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["A", "B"])
def test_slots_and_pages_used_again(name):
    """A pool of eight pages and two slots: sequences come and go; whoever gets a used slot must find the recurrences' states and
    the convolutions' inputs zero, and must not see the keys the pages held before."""
    eng = engine_for(name, "float32", max_tokens=64 * 8, max_slots=2)
    for again in range(3):
        p, q = toks(name, 100 + again, 40 + again), toks(name, 70, 50 + again)
        s1, s2 = eng.cache.open_slot(), eng.cache.open_slot()
        out = eng.step([gi.StepEntry(s1, p, [len(p) - 1]), gi.StepEntry(s2, q, list(range(70)))]).cpu().numpy()
        check(out[:1], plain(name, p).at([len(p) - 1]), "float32", f"use {again}")
        check(out[1:], plain(name, q), "float32", f"use {again}")
        run = eng.decoder([s2])
        extra = toks(name, 3, 90 + again)
        rows = [run.forward(tokens=[x]).cpu().numpy().copy() for x in extra]
        check(np.concatenate(rows, 0), plain(name, q + extra).at(slice(70, None)), "float32", f"use {again}, decoded")
        eng.cache.close_slot(s1)
        eng.cache.close_slot(s2)
    assert eng.cache.free_pages == eng.cache.n_pages


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_sequence_in_a_small_pool(dtype):
    """Windows and chunks of at most 70 positions: a sequence of 900 tokens, the last 300 decoded one by one, lives in a pool of
    five pages, because pages wholly before a window or chunk are given back (and taken again by the same sequence)."""
    cfg = model_cfg(64, 120, [layer("W", win(4, 2, 16, 8, 9, 0.4, 3, rot=8), 24), layer("G", gla(2, 8, 16, 8.0), 24),
                              layer("D", dif(4, 2, 16, 24, 70, 0.3, rot=8))], loop=(0, 2, 2), mult=0.5)
    w = ps.random_weights(cfg, seed=17)
    eng = engine_of(cfg, tensors_of(w, dtype == "bfloat16"), dtype, max_tokens=64 * 5, max_slots=1)
    t = np.random.default_rng(61).integers(0, 120, size=900).tolist()
    s = eng.cache.open_slot()
    rows = [eng.step([gi.StepEntry(s, t[a:a + 50], list(range(50)))]).cpu().numpy() for a in range(0, 600, 50)]
    run = eng.decoder([s])
    rows += [run.forward(tokens=[x]).cpu().numpy().copy() for x in t[600:]]
    eng.cache.close_slot(s)
    assert eng.cache.free_pages == eng.cache.n_pages
    check(np.concatenate(rows, 0), Reference(cfg, w, t), dtype)


# ---- greedy generation through the library's own entry point and command line ---------------------------------------------------
def write_folder(tmp_path, name):
    import json
    from ghost_infer_b200.weights.safetensors_io import save_safetensors
    cfg, w, tensors = made(name)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    save_safetensors(str(folder / "model.safetensors"), tensors)
    return cfg, w, folder


def greedy(cfg, w, prompt, n, clear):
    """The plain implementation's greedy continuation, as far as its choice is clear."""
    seq = list(prompt)
    for _ in range(n):
        logits = ps.forward(cfg, w, seq)[-1]
        order = np.argsort(-logits, kind="stable")
        if logits[order[0]] - logits[order[1]] < clear:
            break
        seq.append(int(order[0]))
    return seq[len(prompt):]


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("A", "bfloat16"), ("B", "float32")])
def test_greedy_generation_through_the_entry_point(tmp_path, name, dtype):
    """`LLM.generate` on a model folder: the scheduler cuts prompts into portions of 16 tokens and decodes two requests at a time."""
    cfg, w, folder = write_folder(tmp_path, name)
    llm = gi.LLM(str(folder), dtype=dtype, max_tokens=64 * 16, max_seq_len=512)
    prompts = [toks(name, n, 80 + i) for i, n in enumerate([3, 30, 11, 75])]
    res = llm.generate(prompts, max_new=6, temperature=0.0, stop_token_ids=(), batch_size=2, max_step_tokens=16)
    followed = 0
    for p, r in zip(prompts, res):
        want = greedy(cfg, w, p, 6, 1e-3 if dtype == "float32" else 0.2)
        followed += len(want)
        assert len(r.tokens) == 6 and r.tokens[:len(want)] == want, f"prompt of {len(p)}: {r.tokens} vs {want}"
    assert followed >= (16 if dtype == "float32" else 2)
    assert llm.cache.free_pages == llm.cache.n_pages


# ---- the replay program as a user runs it ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(tmp_path, dtype):
    """`bin/trace_run` on a model folder: requests whole, tails token by token, and unequal batches decoded together."""
    import json
    import os
    import subprocess
    import sys
    from test_gpu_trace_run import build_trace
    name = "A" if dtype == "bfloat16" else "B"
    cfg, w, folder = write_folder(tmp_path, name)
    reqs, steps = build_trace({"vocab_size": cfg["vocab"]})
    out = tmp_path / "out"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", str(64 * 8)], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                       text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-3000:]
    assert p.stdout.split("\n")[:len(steps)] == [f"done {i}" for i in range(len(steps))]
    place, got, want = {}, [], []
    for s in steps:
        rows = []
        for e in s["entries"]:
            base = place.get(e["id"], 0)
            rows += [plain(name, reqs[e["id"][:2]]).at([base + k]) for k in e["want"]]
            place[e["id"]] = base + len(e["tokens"])
        f = out / f"{s['step']}.f32"
        if rows:
            got.append(np.fromfile(f, dtype="<f4").reshape(-1, cfg["vocab"]))
            want += rows
        else:
            assert not f.exists()
    ref = type("All", (), {})()
    ref.logits, ref.spread = np.concatenate([r.logits for r in want]), np.concatenate([r.spread for r in want])
    check(np.concatenate(got, 0), ref, dtype, "all steps")


# ---- schedules drawn at random ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_drawn_schedules(name):
    """One to four requests of 1 to 200 tokens; every step takes some of the live requests and gives each a portion of 1 to 130
    of its next tokens, so a step holds fresh prompts, portions in mid-sequence and single tokens side by side and some
    requests sit a step out; the places whose logits are wanted are drawn too.  32-bit, so that every row must agree."""
    eng = engine_for(name, "float32", max_tokens=64 * 32, max_seq_len=1024)
    rng = np.random.default_rng(ord(name) + 5)
    rows = 0
    for draw in range(5):
        n_req = int(rng.integers(1, 5))
        lens = [int(rng.integers(1, 200)) for _ in range(n_req)]
        seqs = [toks(name, n, int(rng.integers(1 << 30))) for n in lens]
        refs = [plain(name, t) for t in seqs]
        slots = [eng.cache.open_slot() for _ in seqs]
        done = [0] * n_req
        while any(done[i] < lens[i] for i in range(n_req)):
            live = [i for i in range(n_req) if done[i] < lens[i]]
            pick = [i for i in live if rng.random() < 0.7] or [live[0]]
            entries, wants = [], []
            for i in pick:
                n = int(min(lens[i] - done[i], rng.choice([1, 1, 2, 3, 7, 33, 64, 65, 130])))
                w = sorted(set(int(x) for x in rng.integers(0, n, size=int(rng.integers(0, 3))))) or [n - 1]
                entries.append(gi.StepEntry(slots[i], seqs[i][done[i]:done[i] + n], w))
                wants.append((i, done[i], w))
                done[i] += n
            lg = eng.step(entries).cpu().numpy()
            r = 0
            for i, base, w in wants:
                for x in w:
                    check(lg[r:r + 1], refs[i].at([base + x]), "float32", f"{name} draw {draw}, request {i} of lengths {lens}, place {base + x}")
                    r += 1
            rows += r
        for s in slots:
            eng.cache.close_slot(s)
    assert rows >= 40 and eng.cache.free_pages == eng.cache.n_pages
