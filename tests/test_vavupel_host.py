"""What the Vavupel decoder decides on the host: its configuration, the layers it is built from and the order they run in, the
cache and state it asks for; and the plain implementation's own properties (the oracle is checked apart from the code it judges)."""
import numpy as np
import pytest
import torch

import plain_vavupel as pv
from ghost_infer_b200.cache.sequence_cache import CacheRequest, StateRequest
from ghost_infer_b200.config import ConfigError, architecture_of, parse_config
from ghost_infer_b200.engine.model import Model
from ghost_infer_b200.parts import ModelSpec, PartSpec, ScheduleEntry, looped_schedule

LAT = {"heads": 5, "dim": 10, "rot_dim": 6, "vdim": 12, "kv_rank": 14, "scale": 0.2, "mask": {"size": 9}, "rot": {"base": 3000.0, "dims": 6}}
RET = {"heads": 3, "dim": 8, "vdim": 12, "decay": [0.5, 0.9, 0.99], "rot": {"base": 700.0, "dims": 4}}
MLP = {"kind": "dense", "ff": 28}
CFG = {"architecture": "Vavupel", "width": 40, "vocab": 70, "norm": {"eps": 2e-5}, "logit_softcap": 9.0,
       "embedding": {"scale": 2.5, "bigram": {"buckets": 31, "mul_prev": 11, "mul_cur": 3}},
       "loop": {"start": 1, "stop": 3, "times": 2},
       "layers": [{"type": "retention", "mixer": RET, "mlp": MLP}, {"type": "latent_attention", "mixer": LAT, "mlp": None},
                  {"type": "retention", "mixer": RET, "mlp": MLP}, {"type": "latent_attention", "mixer": LAT, "mlp": MLP}]}


def test_configuration_is_typed_and_checked():
    assert architecture_of(CFG) == "Vavupel"
    cfg = parse_config(CFG)
    assert (cfg.width, cfg.vocab_size, cfg.num_hidden_layers, cfg.norm_eps, cfg.logit_softcap, cfg.embedding_scale) == (40, 70, 4, 2e-5, 9.0, 2.5)
    assert (cfg.pairs.buckets, cfg.pairs.mul_prev, cfg.pairs.mul_cur) == (31, 11, 3)
    assert (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == (1, 3, 2)
    assert cfg.layers[1].mixer.window == 9 and cfg.layers[1].mlp is None and cfg.layers[0].mixer.decay == (0.5, 0.9, 0.99)
    plain = parse_config({k: v for k, v in CFG.items() if k not in ("loop", "logit_softcap", "embedding")})
    assert plain.loop is None and plain.logit_softcap is None and plain.pairs is None and plain.embedding_scale == 1.0
    lay = lambda kind, m, mlp=MLP: {"type": kind, "mixer": m, "mlp": mlp}
    for bad in (dict(CFG, layers=[]), dict(CFG, layers=[lay("mamba2", RET)]),
                dict(CFG, loop={"start": 2, "stop": 2, "times": 1}), dict(CFG, loop={"start": 1, "stop": 5, "times": 1}),
                dict(CFG, loop={"start": 0, "stop": 1, "times": 0}), dict(CFG, logit_softcap=0.0),
                dict(CFG, embedding={"scale": 1.0, "bigram": {"buckets": 0, "mul_prev": 1, "mul_cur": 1}}),
                dict(CFG, layers=[lay("retention", dict(RET, decay=[0.5, 0.9]))]),                             # one decay too few
                dict(CFG, layers=[lay("retention", dict(RET, rot={"base": 10.0, "dims": 10}))]),               # more numbers turn than a head has
                dict(CFG, layers=[lay("latent_attention", dict(LAT, rot={"base": 10.0, "dims": 8}))]),
                dict(CFG, layers=[lay("latent_attention", dict(LAT, rot={"base": 10.0, "dims": 5}))]),
                dict(CFG, layers=[lay("latent_attention", dict(LAT, mask={"size": 0}))]),
                dict(CFG, layers=[lay("latent_attention", {k: v for k, v in LAT.items() if k != "scale"})]),
                dict(CFG, layers=[lay("retention", RET, {"kind": "moe", "ff": 8})]),
                {k: v for k, v in CFG.items() if k != "norm"}, {k: v for k, v in CFG.items() if k != "width"}):
        with pytest.raises(ConfigError):
            parse_config(bad)


def test_layers_are_put_together_from_the_configuration():
    model = Model.from_config_dict(CFG)
    order = [(e.layer, e.inject) for e in model.spec.schedule]
    assert order == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert [(i, p) for i, p in pv.runs(CFG)] == order
    assert [type(l.block).__name__ for l in model.layers] == ["SandwichResidual"] * 4
    assert [type(l.block.mixer).__name__ for l in model.layers] == ["Retention", "LatentAttention", "Retention", "LatentAttention"]
    assert [type(l.block.ffn).__name__ for l in model.layers] == ["Mlp", "NoneType", "Mlp", "Mlp"]
    assert list(model.layers[0].block.extra) == ["mixer_post", "ffn_post"] and list(model.layers[1].block.extra) == ["mixer_post"]
    assert model.injection is not None and model.head.softcap == 9.0 and model.embedding.scale == 2.5
    names = {w.name: tuple(w.shape) for w in model.weight_manifest()}
    assert names == {k: tuple(v.shape) for k, v in pv.random_weights(CFG, 0).items()}
    assert names["loop.in"] == (40, 80) and names["bigram"] == (32, 40) and names["l0.norm1b.alpha"] == () and names["l1.mix.g"] == (5, 40)
    assert "l1.norm2" in model.ignorable_tensors() and "l1.norm2b.alpha" in model.ignorable_tensors()
    bare = Model.from_config_dict({k: v for k, v in CFG.items() if k not in ("loop", "embedding", "logit_softcap")})
    assert bare.injection is None and not any(e.inject for e in bare.spec.schedule) and bare.head.softcap == 0.0
    assert not {"loop.in", "bigram"} & {w.name for w in bare.weight_manifest()}


def test_memory_asked_for():
    """Every pass over the loop has a cache and a state of its own; the embedding keeps a sequence's last token."""
    reqs = Model.from_config_dict(CFG).memory_requests()
    lat = CacheRequest("window", 1, 20, 9, 14, values_in_keys=True)
    ret = StateRequest((3 * 8 * 12,), torch.float32)
    assert [r[1] for r in reqs] == [None, lat, None, lat, None, lat, None]
    assert [r[2] for r in reqs] == [ret, None, ret, None, ret, None, StateRequest((1,), torch.int32)]
    assert all(r[3] is None and r[4] is None for r in reqs)


def test_looped_schedules():
    e = lambda i, inject=False: ScheduleEntry(i, None, inject)
    assert looped_schedule(3, 0, 2, 2, True) == (e(0, True), e(1), e(0, True), e(1), e(2))
    assert looped_schedule(3, 1, 2, 3) == (e(0), e(1), e(1), e(1), e(2))
    assert looped_schedule(2, 2, 2, 1) == (e(0), e(1))
    none = PartSpec("none")
    with pytest.raises(ValueError):           # a schedule that injects in a model without the part
        ModelSpec("x", 8, 8, 8, none, (None,), (e(0, True),), none, none).validate()


# ---- the plain implementation by itself --------------------------------------------------------------------------------
def test_plain_retention_carries_its_state_over_a_cut():
    w = pv.random_weights(CFG, seed=3)
    h = np.random.default_rng(0).standard_normal((30, 40))
    whole, _ = pv.retention(h, np.arange(30), w, "l0.mix.", RET, 1e-5)
    a, st = pv.retention(h[:11], np.arange(11), w, "l0.mix.", RET, 1e-5)
    b, _ = pv.retention(h[11:], np.arange(11, 30), w, "l0.mix.", RET, 1e-5, st)
    assert np.allclose(np.concatenate([a, b]), whole, rtol=1e-12, atol=1e-12)


def test_plain_retention_is_a_decayed_sum_over_earlier_tokens():
    """o_t = sum_j decay^(t - j) (q_t . k_j) v_j / sqrt(dim), q and k rotated: the scan against the sum written out."""
    w = pv.random_weights(CFG, seed=5)
    h = np.random.default_rng(1).standard_normal((12, 40))
    p = "l0.mix."
    q, k = (pv.rotate((h @ w[p + n].T).reshape(12, 3, 8), np.arange(12), 4, 700.0, "half") for n in "qk")
    v = (h @ w[p + "v"].T).reshape(12, 3, 12)
    o = np.zeros((12, 3, 12))
    for a, g in enumerate(RET["decay"]):
        for t in range(12):
            for j in range(t + 1):
                o[t, a] += g ** (t - j) * (q[t, a] @ k[j, a]) / np.sqrt(8.0) * v[j, a]
    z = h @ w[p + "g"].T
    want = ((o / np.sqrt((o ** 2).mean(-1, keepdims=True) + 1e-5)).reshape(12, 36) * z / (1 + np.exp(-z))) @ w[p + "o"].T
    assert np.allclose(pv.retention(h, np.arange(12), w, p, RET, 1e-5)[0], want, rtol=1e-9, atol=1e-10)


def test_plain_window_sink_pairs_and_norm():
    ok = pv.visible(6, 3)
    assert ok[5].tolist() == [False] * 3 + [True] * 3 and ok[1].tolist() == [True, True] + [False] * 4
    assert pv.visible(4).tolist() == np.tril(np.ones((4, 4), dtype=bool)).tolist()
    p = pv.softmax_with_sink(np.array([[0.0, np.log(2.0), -np.inf]]), 0.0)
    assert np.allclose(p, [[0.25, 0.5, 0.0]])                       # the sink takes its share and has no value
    assert pv.bigram_rows([7, 2, 9], {"buckets": 10, "mul_prev": 3, "mul_cur": 4}).tolist() == [10, (21 + 8) % 10, (6 + 36) % 10]
    x = np.array([[0.5, -2.0]])
    w = {"n": np.array([2.0, 3.0]), "n.b": np.array([0.1, 0.2]), "n.alpha": np.array(0.7)}
    assert np.allclose(pv.tanh_norm(x, w, "n"), np.tanh(0.7 * x) * [2.0, 3.0] + [0.1, 0.2])
    assert np.allclose(pv.softcap(np.array([1e9, -1e9, 0.1]), 5.0), [5.0, -5.0, 5.0 * np.tanh(0.02)]) and pv.softcap(3.0, None) == 3.0


def test_plain_far_tokens_reach_only_through_the_recurrence():
    """Latent layers alone: what lies outside every layer's window (and the passes between) changes nothing."""
    cfg = dict(CFG, loop=None, layers=[{"type": "latent_attention", "mixer": dict(LAT, mask={"size": 3}), "mlp": MLP}] * 2)
    w = pv.random_weights(cfg, seed=2)
    t = np.random.default_rng(4).integers(0, 70, size=12).tolist()
    a = pv.forward(cfg, w, t)
    b = pv.forward(cfg, w, [(t[0] + 1) % 70] + t[1:])
    # token 0 reaches position 1 by the pair table, and two more positions per layer
    assert np.allclose(a[6:], b[6:]) and np.abs(a[5] - b[5]).max() > 1e-9
