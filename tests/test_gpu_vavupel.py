"""The Vavupel decoder through the engine, against the plain implementation (`plain_vavupel.py`).

Every test makes its own small configuration and random weights.  The configurations differ from each other in every size and
constant and exercise the values that are easily 1 or equal: one head and many (more than the sixteen one tile holds), keys and
values of different widths, all of a head rotated, a part and none, windows of one position, of a page, of a page and one and
longer than the prompt, loops that start at the first layer, later, and none, a loop of one pass, layers without feed-forward,
embeddings with and without a pair table, capped and uncapped logits, sizes that are multiples of 8 (the tensor-core kernels)
and sizes that are not (the plain ones).  Where random weights would hide a fault the inputs are made: one key whose score
stands out, placed just inside and just outside a window's edge.
"""
import numpy as np
import pytest
import torch

import ghost_infer_b200 as gi
import plain_vavupel as pv

pytestmark = pytest.mark.gpu


def lat(heads, dim, rot_dim, vdim, rank, window, scale, base=10000.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    return dict(m, mask={"size": window}) if window else m


def ret(heads, dim, vdim, rot_dims, base=10000.0, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims},
            "decay": decay or [1.0 - 2.0 ** -(1.0 + 1.7 * h) for h in range(heads)]}


def layer(kind, m, ff=None):
    return {"type": {"L": "latent_attention", "R": "retention"}[kind], "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model_cfg(width, vocab, layers, loop=None, pairs=None, scale=1.0, cap=None, eps=1e-5):
    cfg = {"architecture": "Vavupel", "width": width, "vocab": vocab, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}
    if pairs is not None:
        cfg["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if cap is not None:
        cfg["logit_softcap"] = cap
    return cfg


# multiples of 8 throughout; a loop in the middle
CFG_A = model_cfg(64, 150, [
    layer("R", ret(2, 16, 24, 8, base=900.0), 48),
    layer("L", lat(4, 16, 8, 24, 32, 33, 0.3, base=5000.0), 40),
    layer("R", ret(3, 32, 8, 32)),
    layer("L", lat(8, 24, 16, 16, 40, 70, 0.2, base=700.0), 64),
], loop=(1, 3, 3), pairs=(97, 13, 5), scale=3.0, cap=6.0)
# nothing a multiple of 8, the width not even of 4; the loop starts at the first layer and runs to the last; one head
CFG_B = model_cfg(54, 301, [
    layer("L", lat(3, 6, 4, 5, 11, 1, 0.45, base=77.0), 9),
    layer("R", ret(1, 5, 7, 0)),
    layer("L", lat(1, 10, 2, 6, 13, 65, 0.3), 31),
    layer("R", ret(5, 6, 3, 2, base=50.0), 7),
], loop=(0, 4, 2), pairs=(5, 1000003, 7919), scale=1.0, cap=2.0, eps=3e-6)
# heads as wide as a served model's, more than sixteen of them, a latent wider than 256; a single pass; no pair table, no cap
CFG_C = model_cfg(128, 150, [
    layer("R", ret(2, 128, 64, 64, base=1e6), 128),
    layer("L", lat(20, 64, 32, 32, 96, 64, 0.1, base=250000.0), 96),
    layer("L", lat(2, 32, 48, 40, 272, 100, 0.08), 128),
    layer("R", ret(1, 200, 40, 200)),
], loop=(2, 3, 1), scale=0.5)
# no loop at all; a window longer than any prompt; one pair bucket
CFG_D = model_cfg(40, 90, [
    layer("L", lat(2, 8, 8, 16, 24, 500, 0.3), 24),
    layer("R", ret(2, 8, 8, 8), 24),
    layer("L", lat(6, 8, 8, 8, 8, None, 0.3)),
], pairs=(1, 3, 4), cap=30.0)
CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}
_made = {}


def tensors_of(w, bf16=True):
    out = {k: torch.from_numpy(np.array(v, dtype=np.float32)) for k, v in w.items()}
    return {k: v.to(torch.bfloat16) for k, v in out.items()} if bf16 else out


def made(name):
    if name not in _made:
        cfg = CONFIGS[name]
        w = pv.random_weights(cfg, seed=ord(name))
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
    plain implementation with its intermediate numbers shaken (a head whose read-out nearly vanishes is normed all the same, so
    some positions feel a rounding far more than others)."""

    def __init__(self, cfg, w, tokens):
        self.cfg, self.w, self.tokens = cfg, w, list(tokens)
        self.logits = pv.forward(cfg, w, self.tokens)
        self._spread = None

    @property
    def spread(self):
        if self._spread is None:
            runs_ = [pv.forward(self.cfg, self.w, self.tokens, act=pv.shaken(s)) - self.logits for s in range(8)]
            self._spread = np.max([np.sqrt((r ** 2).mean(axis=1)) for r in runs_], axis=0)
        return self._spread

    def at(self, rows):
        part = object.__new__(Reference)
        part.logits, part._spread = self.logits[rows], self.spread[rows]
        return part


def plain(name, tokens):
    key = (name, tuple(tokens))
    if key not in _plain:
        cfg, w, _ = made(name)
        _plain[key] = Reference(cfg, w, tokens)
    return _plain[key]


def toks(name, n, seed):
    return np.random.default_rng(seed).integers(0, CONFIGS[name]["vocab"], size=n).tolist()


def check(got, ref, dtype, what=""):
    """32-bit: sums of a few hundred terms over a few dozen dependent stages, relative to the largest logit.  bfloat16: per
    position, four times what shaking the plain implementation's intermediate numbers does there (never less than it does
    to the middle position), with room for one position in 25 whose read-out nearly vanished in a way no shaking met; most
    positions must be ones that feel little.  A key one position off, a lost state, a wrong pair or
    a wrong angle moves logits by tens of percent of their spread."""
    got = np.asarray(got, dtype=np.float64)
    assert got.shape == ref.logits.shape, f"{what}: {got.shape} vs {ref.logits.shape}"
    assert np.isfinite(got).all(), f"{what}: non-finite logits"
    scale = max(1.0, float(np.abs(ref.logits).max()))
    err = np.abs(got - ref.logits)
    if dtype == "float32":
        assert err.max() <= 5e-5 * scale, f"{what}: max error {err.max():.3e} (scale {scale:.2f}) at {np.unravel_index(err.argmax(), err.shape)}"
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


# ---- the stream's row kernel, the pair embedding, the cap: against 64-bit torch --------------------------------------------
@pytest.mark.parametrize("rows,width", [(5, 52), (3, 54), (70, 1028), (300, 7), (9, 1), (700, 512)])
def test_the_pass_that_joins_and_reads_the_stream(rows, width):
    from ghost_infer_b200.kernels import ops
    g = torch.Generator(device="cuda:0").manual_seed(rows * 1000 + width)
    rnd = lambda *shape: torch.randn(shape, device="cuda:0", generator=g)
    norm = lambda: (0.3 + float(torch.rand((1,), device="cuda:0", generator=g)), rnd(width), rnd(width))
    plain_norm = lambda u, n: torch.tanh(n[0] * u.double()) * n[1].double() + n[2].double()
    close = lambda a, b: torch.testing.assert_close(a.double(), b, rtol=1e-6, atol=1e-6)
    post, pre = norm(), norm()
    x, y, wide = rnd(rows, width), rnd(rows, width), rnd(rows, 2 * width)
    want = x.double() + plain_norm(y, post)
    x1, y1 = x.clone(), y.clone()
    h = ops.tanh_rows(x1, y1, post, pre, torch.float32, x_out=x1, zero_y=True)
    close(x1, want); close(h, plain_norm(want, pre))
    assert float(y1.abs().max()) == 0.0
    h16 = ops.tanh_rows(x.clone(), y.clone(), post, pre, torch.bfloat16, x_out=x1)
    assert torch.equal(h16, h.bfloat16())
    # the 16-bit path's tanh, over small and large numbers: a few units in the last place, relative
    span = x * torch.logspace(-6, 1.5, rows, device="cuda:0")[:, None]
    unit = (1.0, torch.ones((width,), device="cuda:0"), torch.zeros((width,), device="cuda:0"))
    torch.testing.assert_close(ops.tanh_rows(span, None, None, unit, torch.float32, quick=True).double(), torch.tanh(span.double()), rtol=1.5e-6, atol=0.0)
    close(ops.tanh_rows(x.clone(), y.clone(), post, pre, torch.float32, quick=True), plain_norm(want, pre))
    # rows ready made in the stream's place, the sum handed on as it is
    base, x2 = wide[:, width:], x.clone()
    h = ops.tanh_rows(x2, y, post, None, torch.float32, x_out=x2, base=base)
    close(h, want)
    assert torch.equal(x2, base)
    # two halves of wider rows added; no stream yet; chosen rows only
    x3 = torch.empty_like(x)
    h = ops.tanh_rows(wide[:, :width], base, None, pre, torch.float32, x_out=x3)
    close(x3, wide[:, :width].double() + base.double()); close(h, plain_norm(x3, pre))
    x4 = y.clone()
    assert ops.tanh_rows(None, x4, post, None, None, x_out=x4) is None
    close(x4, plain_norm(y, post))
    pick = torch.tensor([rows - 1, 0, rows // 2, 0], dtype=torch.int32, device="cuda:0")
    close(ops.tanh_rows(x, None, None, pre, torch.float32, rows=pick), plain_norm(x, pre)[pick.long()])
    cap = 3.0
    close(ops.softcap_rows(x.clone() * 4, cap), cap * torch.tanh(x.double() * 4 / cap))


@pytest.mark.parametrize("m,k,width", [(1, 512, 256), (8, 2048, 512), (33, 1000, 260), (64, 4096, 1024)])
def test_pending_sums_are_joined(m, k, width):
    """A one-token step's product leaves the tiles cut between blocks as partial sums; the joining pass adds them, for the
    sublayer's rows and for the stream itself, and never loses them for a later reader."""
    from ghost_infer_b200.kernels import ops
    g = torch.Generator(device="cuda:0").manual_seed(m + k)
    a = torch.randn((m, k), device="cuda:0", generator=g).bfloat16()
    w = (torch.randn((width, k), device="cuda:0", generator=g) / k ** 0.5).bfloat16()
    prod = a.double() @ w.double().T
    x, one = torch.randn((m, width), device="cuda:0", generator=g), torch.ones((width,), device="cuda:0")
    norm = (0.8, one, 0 * one)
    y = ops.as_carrier(torch.zeros((m, width), device="cuda:0"))
    with ops.defer_into(y):
        ops.linear(a, w, out=y, accumulate=True)
    x1 = ops.as_carrier(x.clone())
    h = ops.tanh_rows(x1, y, norm, None, torch.float32, x_out=x1, zero_y=True)
    want = x.double() + torch.tanh(0.8 * prod)
    torch.testing.assert_close(h.double(), want, rtol=1e-5, atol=2e-5)
    assert not ops.has_pending(y) and float(y.as_subclass(torch.Tensor).abs().max()) == 0.0
    with ops.defer_into(x1):
        ops.linear(a, w, out=x1, accumulate=True)
    h = ops.tanh_rows(x1, None, None, norm, torch.float32)          # reads only: the sums are settled into the stream first
    torch.testing.assert_close(h.double(), torch.tanh(0.8 * (want + prod)), rtol=1e-5, atol=2e-5)
    torch.testing.assert_close(x1.as_subclass(torch.Tensor).double(), want + prod, rtol=1e-5, atol=2e-5)


@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(97, 13, 5), (1, 1, 1), (65521, 100003, 99991), (7, 0, 3)])
def test_pairs_across_portions_and_in_a_batch(buckets, mul_prev, mul_cur):
    """Three sequences fed in portions of unequal sizes down to one token, with padding rows between: the token before a
    portion comes from the sequence's state.  The largest products of the multipliers do not fit 32 bits."""
    from ghost_infer_b200.kernels import ops
    vocab, d, scale = 60000, 12, 1.5
    rng = np.random.default_rng(buckets)
    g = torch.Generator(device="cuda:0").manual_seed(1)
    table = torch.randn((vocab, d), device="cuda:0", generator=g)
    pairs = torch.randn((buckets + 1, d), device="cuda:0", generator=g)
    seqs = [rng.integers(vocab - 3000 if mul_prev > 1000 else 0, vocab, size=n).tolist() for n in (23, 9, 300)]
    spec = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    want = [table.double()[torch.tensor(t)] * scale + pairs.double()[torch.from_numpy(pv.bigram_rows(t, spec))] for t in seqs]
    state = torch.full((6, 1), 12345, dtype=torch.int32, device="cuda:0")       # what a slot holds before its first token does not matter
    slot_of, at, got = (2, 0, 4), [0, 0, 0], [[], [], []]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda:0")
    for portion in ((1, 1, 2), (2, 3, 1), (1, 0, 1), (7, 1, 0), (3, 4, 257), (1, 0, 1), (8, 0, 38)):
        step = type("S", (), {})()
        tk, pos, slots, cu, n_seq = [], [], [], [0], 0
        for b, n in enumerate(portion):
            if n:
                tk += seqs[b][at[b]:at[b] + n]; pos += range(at[b], at[b] + n); slots += [slot_of[b]] * n; cu.append(cu[-1] + n); n_seq += 1
        if all(n <= 1 for n in portion):                                         # a recorded step's padding rows
            tk += [0, 0]; pos += [0, 0]; slots += [-1, -1]; cu += [cu[-1] + 1, cu[-1] + 2]; n_seq += 2
        step.tokens, step.positions, step.token_slots, step.cu_seqlens, step.n_seqs = i32(tk), i32(pos), i32(slots), i32(cu), n_seq
        out = ops.embed_pair(table, pairs, step, state, scale, mul_prev, mul_cur)
        o = 0
        for b, n in enumerate(portion):
            got[b].append(out[o:o + n]); o += n; at[b] += n
    for b in range(3):
        torch.testing.assert_close(torch.cat(got[b]).double(), want[b], rtol=1e-6, atol=1e-6)
    assert [int(state[s, 0]) for s in slot_of] == [t[-1] for t in seqs]


# ---- edges made to show: one key whose score stands out, just inside and just outside what a query sees ------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,rank,rot_dim", [(3, 24, 8), (20, 96, 32), (2, 272, 16), (4, 33, 6)])   # keys mode, rows mode, split values, odd sizes
@pytest.mark.parametrize("window", [1, 33, 64, 65, 100, 192, None])
def test_a_key_at_the_windows_edge(dtype, heads, rank, rot_dim, window):
    """Loved rows sit at the first position, on a page's last and first place and in mid-page: the queries just inside and just
    outside their reach show them or not, in a prompt, in portions that end on the edges, and token by token, with a sink and a
    gate per head."""
    from ghost_infer_b200.kernels import ops
    from ghost_infer_b200.cache.sequence_cache import CacheRequest, SequenceCache
    n, H, hd = 300, heads, rank + rot_dim
    rng = np.random.default_rng(3)
    q = np.tile(rng.standard_normal((1, H, hd)), (n, 1, 1)) * 4.0 / np.sqrt(hd)
    rows = rng.standard_normal((n, hd)) * 0.3
    loved = [63, 130, 0, 64][:H]                   # one head each: its other scores stay far below
    for a, p in enumerate(loved):
        rows[p] = q[0, a] * 2.0
    sink, gate = rng.standard_normal(H), rng.standard_normal((n, H))
    mask = pv.visible(n, window)
    ref = np.stack([pv.softmax_with_sink(np.where(mask, (q[:, a] @ rows.T) * 0.5, -np.inf), sink[a]) @ rows[:, :rank] for a in range(H)], axis=1)
    ref = ref * pv.sigmoid(gate)[:, :, None]
    if window:
        for p in loved:
            if 1 < window and p + window < n:      # the oracle itself shows the edge
                assert np.abs(ref[p + window - 1] / pv.sigmoid(gate[p + window - 1])[:, None] - ref[p + window] / pv.sigmoid(gate[p + window])[:, None]).max() > 0.05
    req = CacheRequest("window" if window else "full", 1, hd, window, rank, values_in_keys=True)
    cache = SequenceCache([(0, req, None, None)], max_tokens=64 * 12, max_slots=3, max_seq_len=1024, dtype=dtype, device="cuda:0")
    cache.groups[0].k.fill_(float("nan"))          # whatever no query here sees must not be read
    cache.groups[0].k[:, 0] = 0.0
    dev = lambda a: torch.from_numpy(np.ascontiguousarray(a.reshape(a.shape[0], -1))).to(device="cuda:0", dtype=dtype).contiguous()
    qd, rd, gd, sk = dev(q), dev(rows), dev(gate), torch.from_numpy(sink).to(device="cuda:0", dtype=torch.float32)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda:0")
    w = window or 0
    for cuts in ([n], [2, 131, 130 + w, 131 + w, n] if w and 131 + w < n else [2, 64, 65, n], "tokens"):
        slot = cache.open_slot()
        bounds = list(range(1, n + 1)) if cuts == "tokens" else sorted(set(cuts))
        out, a = [], 0
        for b in bounds:
            cache.reserve([(slot, b)]); cache.sync_tables()
            mem = cache.memory(0)
            pos = torch.arange(a, b, device="cuda:0")
            mem.k[mem.block_table[slot, pos // 64].long(), 0, pos % 64] = rd[a:b]
            step = type("S", (), {})()
            step.is_decode, step.n_seqs, step.max_q_len, step.max_kv_len, step.sm_count = (b - a == 1 and a > 0), 1, b - a, b, 148
            step.cu_seqlens, step.seq_slots, step.seq_pos0, step.seq_lens = i32([0, b - a]), i32([slot]), i32([a]), i32([b])
            lat_ = torch.empty((b - a, H * rank), dtype=dtype, device="cuda:0")
            plan = ops.attn_latent_decode_plan(1, b, 148, H, rank, rot_dim, dtype, window) if step.is_decode else None
            o = ops.attention_latent(qd[a:b].contiguous(), mem, step, H, rank, rot_dim, 0.5, lat_, plan=plan, window=window, sinks=sk, gate=gd[a:b])
            out.append(o.float().cpu().numpy())
            cache.commit(slot, b)
            a = b
        cache.close_slot(slot)
        got = np.concatenate(out, 0).reshape(n, H, rank)
        tol = 3e-5 if dtype == torch.float32 else 0.06
        assert np.abs(got - ref).max() <= tol, f"window {window}, {cuts if cuts == 'tokens' else 'portions'}: {np.abs(got - ref).max():.3e} at {np.unravel_index(np.abs(got - ref).argmax(), got.shape)}"
    assert cache.free_pages == cache.n_pages


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,vdim,rot,adjacent", [(3, 8, 24, 8, False), (2, 64, 64, 32, False), (1, 128, 40, 128, True), (2, 33, 7, 20, False),
                                                        (4, 256, 16, 256, False), (2, 100, 9, 0, False)])
def test_the_rotated_recurrence(dtype, heads, dim, vdim, rot, adjacent):
    """The scan's kernel against the plain sum, state carried over cuts of every kind; one key far back stands out, its head's
    decay close to 1, so that a lost or doubled state shows at the end."""
    from ghost_infer_b200.kernels import ops
    n, base = 260, 3000.0
    rng = np.random.default_rng(dim)
    q, k, v = rng.standard_normal((n, heads, dim)), rng.standard_normal((n, heads, dim)), rng.standard_normal((n, heads, vdim))
    q[200:] = q[200]; k[3] = 3.0 * q[200]
    decay = np.array([0.9995, 0.5, 0.99, 1.0][:heads])
    t16 = lambda a: torch.from_numpy(np.ascontiguousarray(a.reshape(n, -1))).to(device="cuda:0", dtype=dtype)
    qd, kd, vd = t16(q), t16(k), t16(v)
    back = lambda t, w: t.double().cpu().numpy().reshape(n, heads, w)
    layout = "adjacent" if adjacent else "half"
    qr = pv.rotate(back(qd, dim), np.arange(n), rot, base, layout)
    kr = pv.rotate(back(kd, dim), np.arange(n), rot, base, layout) * dim ** -0.5
    v64, S, ref = back(vd, vdim), np.zeros((heads, dim, vdim)), np.zeros((n, heads, vdim))
    for t in range(n):
        S = decay[:, None, None] * S + kr[t][:, :, None] * v64[t][:, None, :]
        ref[t] = np.einsum("hnm,hn->hm", S, qr[t])
    inv = torch.from_numpy(base ** (-2.0 * np.arange(rot // 2) / max(rot, 1))).to("cuda:0", torch.float32)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda:0")
    dc = torch.from_numpy(decay).to("cuda:0", torch.float32)
    packed = torch.cat([qd, kd, vd], dim=1).contiguous()
    qw = heads * dim
    for cuts in ([n], [2, 17, 18, 130, n], [1, 9, 25, 26, 27, n]):
        state = torch.zeros((3, heads * dim * vdim), device="cuda:0")
        out, a = [], 0
        for b in cuts:
            step = type("S", (), {})()
            step.cu_seqlens, step.seq_slots, step.n_seqs = i32([0, b - a]), i32([1]), 1
            table = ops.rope_table(torch.arange(a, b, dtype=torch.int32, device="cuda:0"), inv) if rot else None
            r = packed[a:b]
            out.append(ops.linear_state_rot(r[:, :qw], r[:, qw:2 * qw], r[:, 2 * qw:], state, step, heads, dim, vdim, dc, table, rot, adjacent, dim ** -0.5))
            a = b
        got = torch.cat(out).double().cpu().numpy().reshape(n, heads, vdim)
        assert np.abs(got - ref).max() <= 3e-5 * np.abs(ref).max(), f"cut at {cuts}"
        assert float(state[0].abs().max()) == 0.0 and float(state[2].abs().max()) == 0.0


@pytest.mark.parametrize("rows", [1, 5, 64, 65, 300])
@pytest.mark.parametrize("ff,width", [(48, 64), (320, 256), (7, 54), (4096, 512)])
def test_squared_relu_in_the_products(rows, ff, width):
    from ghost_infer_b200.kernels import ops
    g = torch.Generator(device="cuda:0").manual_seed(rows + ff)
    h = torch.randn((rows, width), device="cuda:0", generator=g)
    w = torch.randn((ff, width), device="cuda:0", generator=g) / width ** 0.5
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        a, b = h.to(dt), w.to(dt)
        want = torch.relu(a.double() @ b.double().T) ** 2
        torch.testing.assert_close(ops.linear_act(a, b, None, "relu2").double(), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("rows,heads,width", [(3, 4, 64), (70, 3, 128), (5, 2, 300), (9, 5, 7), (2, 1, 600)])
@pytest.mark.parametrize("act", ["silu", "sigmoid"])
@pytest.mark.parametrize("weight", [None, "group", "row"])
def test_heads_normed_and_gated(rows, heads, width, act, weight):
    from ghost_infer_b200.kernels import ops
    g = torch.Generator(device="cuda:0").manual_seed(rows + width)
    rnd = lambda *s: torch.randn(s, device="cuda:0", generator=g)
    n = heads * width
    y, wide = rnd(rows, n), rnd(rows, 2 * n)
    w = None if weight is None else rnd(width if weight == "group" else n)
    gate = wide[:, n:]
    u = y.double().view(rows, heads, width)
    ref = (u / torch.sqrt((u ** 2).mean(-1, keepdim=True) + 1e-5)).view(rows, n)
    if w is not None:
        ref = ref * (w.double().repeat(heads) if weight == "group" else w.double())
    ref = ref * torch.sigmoid(gate.double()) * (gate.double() if act == "silu" else 1.0)
    torch.testing.assert_close(ops.norm_gate(y, gate, w, width, 1e-5, act, torch.float32).double(), ref, rtol=2e-5, atol=2e-5)
    g16 = gate.bfloat16()
    got = ops.norm_gate(y, g16, w, width, 1e-5, act, torch.bfloat16)
    assert torch.equal(got, ops.norm_gate(y, g16.float(), w, width, 1e-5, act, torch.float32).bfloat16())


# ---- the arrangement and the loop by themselves ------------------------------------------------------------------------
def test_a_sandwich_of_other_norms():
    """The block with RMS norms, which cannot join on the way: the same sums, one operation after the other."""
    from ghost_infer_b200.parts import FeedForward, Mixer, Runtime, lookup
    d, T = 48, 9
    g = torch.Generator(device="cuda:0").manual_seed(2)
    rt = Runtime(torch.device("cuda:0"), torch.float32)
    ws = {f"n{i}": torch.rand((d,), device="cuda:0", generator=g) + 0.5 for i in range(4)}
    norms = []
    for i in range(4):
        norms.append(lookup("norm", "rmsnorm")({"size": d, "eps": 1e-5, "tensor_names": {"weight": ""}}, f"n{i}"))
        norms[-1].bind(ws, rt)
    a, b = (torch.randn((d, d), device="cuda:0", generator=g) / d ** 0.5 for _ in range(2))

    class Mix(Mixer):
        def forward(self, h, residual, step, memory):
            residual += h @ a.T

    class Ffn(FeedForward):
        def forward(self, h, residual, step):
            residual += h @ b.T

    block = lookup("block", "sandwich_residual")(norms[0], Mix({}), norms[2], Ffn({}), mixer_post=norms[1], ffn_post=norms[3])
    step = type("S", (), {"shared": {}, "next_reader": None})()
    x = torch.randn((T, d), device="cuda:0", generator=g)
    rms = lambda u, w: u / torch.sqrt((u ** 2).mean(-1, keepdim=True) + 1e-5) * w.double()
    want = x.double()
    for m, n1, n2 in ((a, "n0", "n1"), (b, "n2", "n3")):
        want = want + rms(rms(want, ws[n1]) @ m.double().T, ws[n2])
    block.forward(x, step, None)
    torch.testing.assert_close(x.double(), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("starts", [True, False])
def test_injection_with_and_without_a_writer_that_helps(dtype, starts):
    from ghost_infer_b200.kernels import ops
    from ghost_infer_b200.parts import Runtime, lookup
    d, T = 64, 6
    g = torch.Generator(device="cuda:0").manual_seed(3)
    w = (torch.randn((d, 2 * d), device="cuda:0", generator=g) / (2 * d) ** 0.5).bfloat16().float()
    part = lookup("injection", "input_injection")({"hidden_size": d}, "loop.in")
    assert part.weights()[0].name == "loop.in"
    part.bind({"loop.in": w}, Runtime(torch.device("cuda:0"), getattr(torch, dtype)))
    x0, x1, x2 = (torch.randn((T, d), device="cuda:0", generator=g) for _ in range(3))
    want = lambda x: torch.cat([x, x0], 1).double() @ w.double().T
    tol = 1e-5 if dtype == "float32" else 2e-2
    step = type("S", (), {"shared": {}, "next_reader": None})()
    x = ops.as_carrier(x0.clone())
    part.begin(x, step, starts)
    part.forward(x, step)                                    # the first pass: the stream is still the embedding's output
    ops.settle(x)
    torch.testing.assert_close(x.as_subclass(torch.Tensor).double(), want(x0), rtol=tol, atol=tol)
    for later in (x1, x2):                                    # nobody prepared the stream: the part does it itself
        x.as_subclass(torch.Tensor).copy_(later)
        part.forward(x, step)
        ops.settle(x)
        torch.testing.assert_close(x.as_subclass(torch.Tensor).double(), want(later), rtol=tol, atol=tol)


# ---- each mechanism alone: one- and two-layer models ------------------------------------------------------------------
ALONE = {
    "latent": ([layer("L", lat(3, 6, 4, 5, 12, 7, 0.4))], {}),
    "latent_one_head_window_one": ([layer("L", lat(1, 4, 2, 4, 8, 1, 0.5))], {}),
    "latent_rotated_part_wide": ([layer("L", lat(2, 2, 16, 8, 16, 33, 0.3, base=50.0))], {}),
    "latent_window_longer_than_the_prompt": ([layer("L", lat(2, 8, 8, 8, 16, 500, 0.3))], {}),
    "retention": ([layer("R", ret(3, 6, 9, 4))], {}),
    "retention_unrotated_one_head": ([layer("R", ret(1, 4, 4, 0, decay=[1.0]))], {}),
    "retention_no_memory": ([layer("R", ret(2, 4, 12, 4, decay=[0.0, 0.25]))], {}),
    "retention_widest_keys": ([layer("R", ret(1, 256, 4, 256))], {}),
    "feed_forward": ([layer("R", ret(1, 4, 4, 2), 30)], {}),
    "pairs": ([layer("L", lat(2, 4, 4, 4, 8, 3, 0.4), 8)], {"pairs": (11, 7, 3), "scale": 4.0}),
    "loop_over_everything": ([layer("R", ret(2, 4, 4, 4), 8), layer("L", lat(2, 4, 4, 4, 8, 9, 0.4), 8)], {"loop": (0, 2, 3)}),
    "loop_of_one_layer_at_the_end": ([layer("R", ret(2, 4, 4, 4), 8), layer("L", lat(2, 4, 4, 4, 8, 9, 0.4))], {"loop": (1, 2, 4)}),
    "loop_of_one_pass": ([layer("R", ret(2, 4, 4, 4), 8)], {"loop": (0, 1, 1)}),
    "cap": ([layer("R", ret(2, 4, 4, 4), 8)], {"cap": 0.7}),
}


@pytest.mark.parametrize("which", sorted(ALONE))
@pytest.mark.parametrize("width", [48, 45])
def test_each_mechanism_alone(which, width):
    layers, opts = ALONE[which]
    cfg = model_cfg(width, 90, layers, **opts)
    w = pv.random_weights(cfg, seed=11)
    eng = engine_of(cfg, tensors_of(w, False), "float32", max_tokens=256, max_seq_len=256)
    t = np.random.default_rng(5).integers(0, 90, size=70).tolist()
    ref = Reference(cfg, w, t)
    check(run_whole(eng, t), ref, "float32", which)
    check(prompt_then_tokens(eng, t, 30), ref, "float32", which + ", decoded")


def test_the_stream_after_every_layer_run():
    """Through a loop: what the stream holds after each run of a layer (where a pass follows, what is handed to it)."""
    from ghost_infer_b200.kernels import ops
    cfg, w, tensors = made("A")
    eng = engine_of(cfg, tensors, "float32")
    seen = []
    for lay in eng.model.layers:
        def spied(x, step, memory, run=lay.block.forward):
            run(x, step, memory)
            left = x.__dict__.get("_gi_handed")
            raw = x.as_subclass(torch.Tensor)
            seen.append((left[1] if left is not None and left[0] is eng.model.injection else raw).double().cpu().numpy())
        lay.block.forward = spied
    t = toks("A", 50, 3)
    run_whole(eng, t)
    _, after = pv.forward(cfg, w, t, return_layers=True)
    assert len(seen) == len(after) == 8
    for i, (got, ref) in enumerate(zip(seen, after)):
        assert np.abs(got - ref).max() <= 5e-5 * np.abs(ref).max(), f"after run {i}"


# ---- whole prompts, decoding, portions, batches -----------------------------------------------------------------------
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
    t = toks(name, 150, 21)          # decoded across the page borders at 64 and 128 and out of every window
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
    """One step holds the second portion of one request and the whole of another: positions and pairs count from 0 in each."""
    eng = engine_for("A", "float32")
    a, b = toks("A", 120, 61), toks("A", 40, 62)
    s1, s2 = eng.cache.open_slot(), eng.cache.open_slot()
    r0 = eng.step([gi.StepEntry(s1, a[:50], list(range(50)))]).cpu().numpy()
    r1 = eng.step([gi.StepEntry(s2, b, list(range(40))), gi.StepEntry(s1, a[50:110], list(range(60)))]).cpu().numpy()
    r2 = eng.step([gi.StepEntry(s1, a[110:], list(range(10)))]).cpu().numpy()
    eng.cache.close_slot(s1); eng.cache.close_slot(s2)
    check(np.concatenate([r0, r1[40:], r2], 0), plain("A", a), "float32", "under way")
    check(r1[:40], plain("A", b), "float32", "fresh")


# ---- pages and slots given back and used again ---------------------------------------------------------------------
@pytest.mark.parametrize("name", ["A", "B"])
def test_slots_and_pages_used_again(name):
    """A pool of six pages and two slots: sequences come and go; whoever gets a used slot must find the recurrences' states zero
    and no token before its first, and must not see the latents the pages held before."""
    eng = engine_for(name, "float32", max_tokens=64 * 6, max_slots=2)
    for round_ in range(3):
        p, q = toks(name, 100 + round_, 40 + round_), toks(name, 70, 50 + round_)
        s1, s2 = eng.cache.open_slot(), eng.cache.open_slot()
        out = eng.step([gi.StepEntry(s1, p, [len(p) - 1]), gi.StepEntry(s2, q, list(range(70)))]).cpu().numpy()
        check(out[:1], plain(name, p).at([len(p) - 1]), "float32", f"round {round_}")
        check(out[1:], plain(name, q), "float32", f"round {round_}")
        run = eng.decoder([s2])
        extra = toks(name, 3, 90 + round_)
        rows = [run.forward(tokens=[x]).cpu().numpy().copy() for x in extra]
        check(np.concatenate(rows, 0), plain(name, q + extra).at(slice(70, None)), "float32", f"round {round_}, decoded")
        eng.cache.close_slot(s1)
        eng.cache.close_slot(s2)
    assert eng.cache.free_pages == eng.cache.n_pages


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_sequence_in_a_small_pool(dtype):
    """Windows of at most 70 positions: a sequence of 900 tokens, the last 300 decoded one by one, lives in a pool of four pages,
    because pages wholly before a window are given back (and taken again by the same sequence)."""
    cfg = model_cfg(64, 120, [layer("L", lat(2, 16, 8, 8, 16, 9, 0.4), 24), layer("R", ret(2, 8, 16, 8), 24), layer("L", lat(4, 16, 8, 8, 24, 70, 0.3))],
                    loop=(0, 2, 2), pairs=(50, 3, 7))
    w = pv.random_weights(cfg, seed=17)
    eng = engine_of(cfg, tensors_of(w, dtype == "bfloat16"), dtype, max_tokens=64 * 4, max_slots=1)
    t = np.random.default_rng(61).integers(0, 120, size=900).tolist()
    s = eng.cache.open_slot()
    rows = [eng.step([gi.StepEntry(s, t[a:a + 50], list(range(50)))]).cpu().numpy() for a in range(0, 600, 50)]
    run = eng.decoder([s])
    rows += [run.forward(tokens=[x]).cpu().numpy().copy() for x in t[600:]]
    eng.cache.close_slot(s)
    assert eng.cache.free_pages == eng.cache.n_pages
    check(np.concatenate(rows, 0), Reference(cfg, w, t), dtype)


# ---- greedy generation through the library's own entry point ---------------------------------------------------------------
@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("A", "bfloat16"), ("B", "float32")])
def test_greedy_generation_through_the_entry_point(tmp_path, name, dtype):
    """`LLM.generate` on a model folder: the scheduler cuts prompts into portions of 16 tokens and decodes two requests at a
    time; every greedy token is the plain implementation's, as long as that one's choice is clear."""
    import json
    from ghost_infer_b200.weights.safetensors_io import save_safetensors
    cfg, w, tensors = made(name)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    save_safetensors(str(folder / "model.safetensors"), tensors)
    llm = gi.LLM(str(folder), dtype=dtype, max_tokens=64 * 16, max_seq_len=512)
    prompts = [toks(name, n, 80 + i) for i, n in enumerate([3, 30, 11, 75])]
    res = llm.generate(prompts, max_new=6, temperature=0.0, stop_token_ids=(), batch_size=2, max_step_tokens=16)
    clear, followed = (1e-3 if dtype == "float32" else 0.2), 0
    for p, r in zip(prompts, res):
        seq = list(p)
        for _ in range(6):
            logits = pv.forward(cfg, w, seq)[-1]
            order = np.argsort(-logits, kind="stable")
            if logits[order[0]] - logits[order[1]] < clear:
                break
            seq.append(int(order[0]))
        want = seq[len(p):]
        followed += len(want)
        assert len(r.tokens) == 6 and r.tokens[:len(want)] == want, f"prompt of {len(p)}: {r.tokens} vs {want}"
    assert followed >= (16 if dtype == "float32" else 2)
    assert llm.cache.free_pages == llm.cache.n_pages


# ---- the replay program as a user runs it ----------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(tmp_path, dtype):
    """`bin/trace_run` on a model folder: requests whole, tails token by token, and unequal batches decoded together."""
    import json
    import os
    import subprocess
    import sys
    from ghost_infer_b200.weights.safetensors_io import save_safetensors
    from test_gpu_trace_run import build_trace
    name = "A" if dtype == "bfloat16" else "B"
    cfg, w, tensors = made(name)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    save_safetensors(str(folder / "model.safetensors"), tensors)
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
    ref = object.__new__(Reference)
    ref.logits, ref._spread = np.concatenate([r.logits for r in want]), np.concatenate([r.spread for r in want])
    check(np.concatenate(got, 0), ref, dtype, "all steps")


# ---- schedules drawn at random ------------------------------------------------------------------------------------------
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
