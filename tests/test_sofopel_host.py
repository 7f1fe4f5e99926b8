"""What the Sofopel decoder decides on the host: its configuration, the layers it is built from and the order they run in, the
cache and state it asks for; and the plain implementation's own properties (the oracle is checked apart from the code it judges)."""
import math

import numpy as np
import pytest
import torch

import plain_sofopel as ps
from ghost_infer_b200.cache.sequence_cache import CacheRequest, StateRequest
from ghost_infer_b200.config import ConfigError, architecture_of, parse_config
from ghost_infer_b200.engine.model import Model
from ghost_infer_b200.parts import ScheduleEntry, WeightSpec
from ghost_infer_b200.parts.rope import rotary_inv_freq
from ghost_infer_b200.weights.loader import WeightsError, load_model_tensors
from ghost_infer_b200.weights.safetensors_io import save_safetensors

YARN = {"factor": 3.0, "original": 60, "fast": 8.0, "slow": 1.5}
DIF = {"heads": 6, "kv_heads": 2, "dim": 6, "vdim": 10, "scale": 0.4, "diff": 0.2, "conv": 3, "mask": {"size": 9}, "rot": {"base": 3000.0, "dims": 4}}
WIN = {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 12, "scale": 0.3, "mask": {"size": 7, "keep_first": 2},
       "rot": {"base": 700.0, "dims": 8, "scaling": YARN}}
GLA = {"heads": 3, "dim": 8, "vdim": 12, "tau": 5.0}
MLP = {"kind": "dense", "ff": 28, "limit": 1.5}
CFG = {"architecture": "Sofopel", "width": 40, "vocab": 70, "norm": {"eps": 2e-5}, "embedding": {"scale": 2.5}, "residual_mult": 0.6,
       "loop": {"start": 1, "stop": 3, "times": 2},
       "layers": [{"type": "attention", "mixer": DIF, "mlp": MLP}, {"type": "gla", "mixer": GLA, "mlp": None},
                  {"type": "attention_2", "mixer": WIN, "mlp": MLP}, {"type": "gla", "mixer": GLA, "mlp": MLP}]}


def test_configuration_is_typed_and_checked():
    assert architecture_of(CFG) == "Sofopel"
    cfg = parse_config(CFG)
    assert (cfg.width, cfg.vocab_size, cfg.num_hidden_layers, cfg.norm_eps, cfg.embedding_scale, cfg.residual_mult) == (40, 70, 4, 2e-5, 2.5, 0.6)
    assert (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == (1, 3, 2)
    d, g, w = cfg.layers[0].mixer, cfg.layers[1].mixer, cfg.layers[2].mixer
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.scale, d.diff, d.conv, d.chunk, d.rot.dims) == (6, 2, 6, 10, 0.4, 0.2, 3, 9, 4)
    assert (w.window, w.keep_first, w.rot.scaling.factor, w.rot.scaling.slow) == (7, 2, 3.0, 1.5)
    assert (g.heads, g.dim, g.vdim, g.tau) == (3, 8, 12, 5.0) and cfg.layers[1].mlp is None and cfg.layers[0].mlp.limit == 1.5
    lay = lambda kind, m, mlp=MLP: {"type": kind, "mixer": m, "mlp": mlp}
    without = lambda m, *keys: {k: v for k, v in m.items() if k not in keys}
    plain = parse_config(dict(without(CFG, "loop", "embedding", "residual_mult"),
                              layers=[lay("attention", without(DIF, "mask", "rot", "conv")), lay("attention_2", without(WIN, "mask", "rot"))]))
    assert plain.loop is None and plain.embedding_scale == 1.0 and plain.residual_mult == 1.0
    assert plain.layers[0].mixer.chunk is None and plain.layers[0].mixer.rot is None and plain.layers[0].mixer.conv == 0
    assert plain.layers[1].mixer.window is None and plain.layers[1].mixer.keep_first == 0
    for bad in (dict(CFG, layers=[]), dict(CFG, layers=[lay("mamba2", GLA)]), dict(CFG, loop={"start": 2, "stop": 2, "times": 1}),
                dict(CFG, loop={"start": 1, "stop": 5, "times": 1}), dict(CFG, loop={"start": 0, "stop": 1, "times": 0}),
                dict(CFG, layers=[lay("gla", dict(GLA, tau=0.0))]), dict(CFG, layers=[lay("gla", without(GLA, "tau"))]),
                dict(CFG, layers=[lay("attention", dict(DIF, kv_heads=4))]), dict(CFG, layers=[lay("attention", without(DIF, "diff"))]),
                dict(CFG, layers=[lay("attention", dict(DIF, rot={"base": 10.0, "dims": 8}))]),
                dict(CFG, layers=[lay("attention", dict(DIF, rot={"base": 10.0, "dims": 3}))]),
                dict(CFG, layers=[lay("attention", dict(DIF, mask={"size": 0}))]), dict(CFG, layers=[lay("attention", dict(DIF, conv=0))]),
                dict(CFG, layers=[lay("attention_2", dict(WIN, mask={"size": 4, "keep_first": -1}))]),
                dict(CFG, layers=[lay("attention_2", dict(WIN, rot=dict(WIN["rot"], scaling=without(YARN, "fast"))))]),
                dict(CFG, layers=[lay("attention_2", without(WIN, "scale"))]), dict(CFG, layers=[lay("gla", GLA, {"kind": "moe", "ff": 8})]),
                dict(CFG, layers=[lay("gla", GLA, {"kind": "dense", "ff": 8})]), dict(CFG, layers=[lay("gla", GLA, dict(MLP, limit=0.0))]),
                without(CFG, "norm"), without(CFG, "width")):
        with pytest.raises(ConfigError):
            parse_config(bad)


def test_layers_are_put_together_from_the_configuration():
    model = Model.from_config_dict(CFG)
    assert [e.layer for e in model.spec.schedule] == ps.runs(CFG) == [0, 1, 2, 1, 2, 3]
    assert all(e == ScheduleEntry(e.layer) for e in model.spec.schedule)
    assert [type(l.block).__name__ for l in model.layers] == ["ParallelResidual"] * 4
    assert [type(l.block.mixer).__name__ for l in model.layers] == ["DifferentialAttention", "GatedLinearAttention", "HeadNormedAttention", "GatedLinearAttention"]
    assert [type(l.block.ffn).__name__ for l in model.layers] == ["SwiGlu", "NoneType", "SwiGlu", "SwiGlu"]
    assert all(l.block.params["scale"] == 0.6 and l.block.ffn_norm is None and l.block.first_reader() is l.block.mixer_norm for l in model.layers)
    ffn, win, dif = model.layers[0].block.ffn, model.layers[2].block.mixer, model.layers[0].block.mixer
    assert (ffn.activation, ffn.limit, ffn.alpha) == ("clamped", 1.5, 1.702) and model.embedding.scale == 2.5
    assert win.zero_sink and not win.has_sink and win.keep_first == 2 and win.rotary.magnitude == pytest.approx(0.1 * math.log(3.0) + 1.0)
    assert dif.adjacent and not win.adjacent and dif.key_width == 12
    names = {w.name: tuple(w.shape) for w in model.weight_manifest()}
    assert names == {k: tuple(v.shape) for k, v in ps.random_weights(CFG, 0, rank=16).items()}
    assert names["l0.mix.q.conv"] == (72, 3) and names["l0.mix.lq1"] == (6,) and names["l2.mix.g"] == (4, 40) and "l2.mix.sink" not in names
    no_conv = Model.from_config_dict(dict(CFG, layers=[dict(CFG["layers"][0], mixer={k: v for k, v in DIF.items() if k != "conv"})], loop=None))
    assert not any(w.name.endswith(".conv") for w in no_conv.weight_manifest()) and no_conv.memory_requests()[0][2] is None


def test_memory_asked_for():
    """Every pass over the loop has a cache and a state of its own; a differential layer has both."""
    reqs = Model.from_config_dict(CFG).memory_requests()
    dif, win = CacheRequest("chunk", 2, 12, 9, 10), CacheRequest("window", 2, 10, 7, 12, keep_first=2)
    conv, gla = StateRequest((2 * (72 + 24 + 20),), torch.float32), StateRequest((3 * 8 * 12,), torch.float32)
    assert [r[1] for r in reqs] == [dif, None, win, None, win, None]
    assert [r[2] for r in reqs] == [conv, gla, None, gla, None, gla]
    assert all(r[3] is None and r[4] is None for r in reqs)


def test_a_size_that_only_the_file_knows(tmp_path):
    """The width between the decay's two matrices comes from the file, layer by layer; every other shape must fit."""
    model = Model.from_config_dict(CFG)
    free = {w.name: w.free for w in model.weight_manifest() if w.free}
    assert free == {"l1.mix.a1": (0,), "l1.mix.a2": (1,), "l3.mix.a1": (0,), "l3.mix.a2": (1,)}
    tensors = {k: torch.from_numpy(v.astype(np.float32)) for k, v in ps.random_weights(CFG, 1, rank={1: 3, 3: 7}).items()}
    save_safetensors(str(tmp_path / "model.safetensors"), tensors)
    got = load_model_tensors(str(tmp_path), model.weight_manifest())
    assert tuple(got["l1.mix.a1"].shape) == (3, 40) and tuple(got["l3.mix.a2"].shape) == (24, 7)
    model.bind(got, "float32", "cpu")
    assert [l.block.mixer.rank for l in model.layers if hasattr(l.block.mixer, "rank")] == [3, 7]
    for wrong, shape in (("l1.mix.a1", (3, 41)), ("l1.mix.a2", (23, 3)), ("l1.mix.q", (23, 40)), ("l1.mix.a1", (3,))):
        save_safetensors(str(tmp_path / "model.safetensors"), dict(tensors, **{wrong: torch.zeros(shape)}))
        with pytest.raises(WeightsError):
            load_model_tensors(str(tmp_path), model.weight_manifest())
    with pytest.raises(ValueError):            # the two matrices must agree
        Model.from_config_dict(CFG).bind(dict(tensors, **{"l1.mix.a2": torch.zeros((24, 4))}), "float32", "cpu")
    assert WeightSpec("x", (2, 3)).free == ()


def test_scaled_frequencies():
    for dims, base, sc in ((8, 700.0, YARN), (48, 10000.0, {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                           (2, 9.0, {"factor": 2.0, "original": 7, "fast": 40.0, "slow": 39.0})):
        want, magnitude = ps.frequencies(dims, base, sc)
        got = rotary_inv_freq(dims, base, dict(sc, rope_type="yarn")).double().numpy()
        assert np.allclose(got, want, rtol=1e-6) and magnitude == pytest.approx(0.1 * math.log(sc["factor"]) + 1.0)


# ---- the plain implementation by itself --------------------------------------------------------------------------------
def test_plain_gated_linear_attention_carries_its_state_over_a_cut():
    w = ps.random_weights(CFG, seed=3)
    h = np.random.default_rng(0).standard_normal((30, 40))
    whole, _ = ps.gated_linear_attention(h, w, "l1.mix.", GLA, 1e-5)
    a, st = ps.gated_linear_attention(h[:11], w, "l1.mix.", GLA, 1e-5)
    b, _ = ps.gated_linear_attention(h[11:], w, "l1.mix.", GLA, 1e-5, st)
    assert np.allclose(np.concatenate([a, b]), whole, rtol=1e-12, atol=1e-12)


def test_plain_gated_linear_attention_is_a_decayed_sum_over_earlier_tokens():
    """o_t = sum_j sum_c q_tc k_jc (prod of the channel's decays after j) v_j / sqrt(dim): the scan against the sum written out."""
    w = ps.random_weights(CFG, seed=5)
    h = np.random.default_rng(1).standard_normal((12, 40))
    p = "l1.mix."
    q, k = ((h @ w[p + n].T).reshape(12, 3, 8) for n in "qk")
    v = (h @ w[p + "v"].T).reshape(12, 3, 12)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = (1.0 / (1.0 + np.exp(-z)) ** (1.0 / 5.0)).reshape(12, 3, 8)
    o = np.zeros((12, 3, 12))
    for t in range(12):
        for j in range(t + 1):
            through = alpha[j + 1:t + 1].prod(axis=0)
            o[t] += (q[t] * k[j] * through).sum(-1)[:, None] / np.sqrt(8.0) * v[j]
    g = h @ w[p + "g"].T
    o = o / np.sqrt((o ** 2).mean(-1, keepdims=True) + 1e-5) * w[p + "norm"]
    want = (o.reshape(12, 36) * g / (1 + np.exp(-g))) @ w[p + "o"].T
    assert np.allclose(ps.gated_linear_attention(h, w, p, GLA, 1e-5)[0], want, rtol=1e-9, atol=1e-10)


def test_plain_masks_softmax_convolution_and_maps():
    ok = ps.window_and_first(7, 3, 2)
    assert ok[6].tolist() == [True, True, False, False, True, True, True] and ok[1].tolist() == [True, True] + [False] * 5
    assert ps.same_chunk(5, 2).tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    assert np.allclose(ps.softmax_plus_one(np.array([[0.0, np.log(2.0), -np.inf]])), [[0.25, 0.5, 0.0]])
    u = np.arange(1.0, 5.0)[:, None]
    assert ps.short_conv(u, np.array([[100.0, 10.0, 1.0]]))[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0]
    w = {"lq1": np.array([1.0, 2.0]), "lk1": np.array([0.5, 0.0]), "lq2": np.array([1.0, 1.0]), "lk2": np.array([0.0, -1.0])}
    assert ps.map_weight(w, "", 0.2) == pytest.approx(np.exp(0.5) - np.exp(-1.0) + 0.2)
    o = ps.difference_of_maps(np.array([3.0, 5.0]), np.array([1.0, 2.0]), 2.0, 0.25, 0.0)
    assert np.allclose(o, np.array([1.0, 1.0]) * 0.75)


def test_plain_far_tokens_reach_only_through_what_keeps_them():
    """Window layers without kept positions: what lies outside every layer's window changes nothing; kept positions bring it in."""
    w0 = dict(WIN, mask={"size": 3})
    for keep, far in ((0, False), (1, True)):
        m = dict(w0, mask={"size": 3, "keep_first": keep})
        cfg = dict(CFG, loop=None, layers=[{"type": "attention_2", "mixer": m, "mlp": MLP}] * 2)
        w = ps.random_weights(cfg, seed=2)
        t = np.random.default_rng(4).integers(0, 70, size=12).tolist()
        a, b = ps.forward(cfg, w, t), ps.forward(cfg, w, [(t[0] + 1) % 70] + t[1:])
        assert (np.abs(a[6:] - b[6:]).max() > 1e-9) == far and np.abs(a[4] - b[4]).max() > 1e-9
