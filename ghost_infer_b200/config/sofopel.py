"""Typed configuration of the Sofopel decoder, read from config.json, and the layers it is made of.

A layer of a Sofopel model norms the stream once; its mixer and its feed-forward both read that norm, and their sum, times
`residual_mult`, joins the stream: x += residual_mult * (mixer(h) + ff(h)), h = rms(x).  With `loop` = {`start`, `stop`, `times`}
the layers start .. stop - 1 run `times` times in a row on the same weights, each pass with a cache or state of its own.
`layers[i].type` names the mixer, `layers[i].mixer` gives its sizes:

* "attention": differential attention: every head has two maps (queries and keys of `dim` numbers each, neighbouring pairs of
  the first `rot.dims` turn) over one value of `vdim`, and gives the first map's output less a learned share of the second's
  (`diff` enters it), normed; queries, keys and values pass a causal convolution over `conv` tokens first; a position sees its
  own chunk of `mask.size` positions;
* "attention_2": grouped-query attention with per-head norms of queries and keys, pairs half of `rot.dims` apart turned (`rot.
  scaling`: YaRN), a window of `mask.size` positions that keeps the first `mask.keep_first`, one added to the softmax's
  denominator, one sigmoid gate per head;
* "gla": gated linear attention: a matrix of state per head that decays per key channel by sigmoid(.)^(1 / `tau`).

The feed-forward (`mlp.kind` "dense") is a gated one with halves clamped to `mlp.limit`; `mlp` null: none.  The embedding is
multiplied by `embedding.scale`; every norm of the stream is an RMS norm with `norm.eps`; the head is a matrix of its own.
Nothing about a model lives in code: sizes, counts, constants and the order of layers come from config.json; the one size it
does not hold, the width between the decay's two matrices, comes from the weights file.

Tensors: "embed", "l<i>.norm1", "l<i>.mix.*", "l<i>.mlp.{gate,up,down}", "final.norm", "head".
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..parts.spec import LayerSpec, ModelSpec, PartSpec, looped_schedule
from .errors import ConfigError

ARCHITECTURE = "Sofopel"
# rotary angles are formed from the position itself: no length the design was trained for is written anywhere
NO_POSITION_LIMIT = 1 << 20
# fixed by the design: what the gate is multiplied by inside its sigmoid
GATE_ALPHA = 1.702


def _need(d: Any, key: str, where: str):
    if not isinstance(d, Mapping) or key not in d or d[key] is None:
        raise ConfigError(f"config.json of {ARCHITECTURE}: missing key \"{key}\" in {where}")
    return d[key]


def _int(d: Any, key: str, where: str, least: int = 1) -> int:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or int(v) != v or int(v) < least:
        raise ConfigError(f"config.json of {ARCHITECTURE}: \"{key}\" in {where} must be an integer >= {least}, got {v!r}")
    return int(v)


def _num(d: Any, key: str, where: str, positive: bool = False) -> float:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and not v > 0):
        raise ConfigError(f"config.json of {ARCHITECTURE}: \"{key}\" in {where} must be a {'positive ' if positive else ''}number, got {v!r}")
    return float(v)


@dataclass(frozen=True)
class Yarn:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    scaling: Optional[Yarn] = None


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class DifferentialMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    conv: int                      # 0: none
    rot: Optional[Rotation]
    chunk: Optional[int]


@dataclass(frozen=True)
class WindowMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Rotation]
    window: Optional[int]
    keep_first: int


@dataclass(frozen=True)
class GlaMixer:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class DenseMlp:
    ff: int
    limit: float


@dataclass(frozen=True)
class SofopelLayer:
    type: str
    mixer: Any
    mlp: Optional[DenseMlp]


def _rotation(m: Any, where: str, most: int) -> Optional[Rotation]:
    if not isinstance(m, Mapping) or m.get("rot") is None:
        return None
    r, where = m["rot"], where + ".rot"
    dims = _int(r, "dims", where, least=0)
    if dims % 2 or dims > most:
        raise ConfigError(f"config.json of {ARCHITECTURE}: {where}: {dims} rotated numbers must be even and at most {most}")
    base = _num(r, "base", where, positive=True)
    scaling = None
    if r.get("scaling") is not None:
        s, sw = r["scaling"], where + ".scaling"
        scaling = Yarn(*(_num(s, k, sw, positive=True) for k in ("factor", "original", "fast", "slow")))
        if base == 1.0:
            raise ConfigError(f"config.json of {ARCHITECTURE}: {where}: a scaled rotation needs a base other than 1")
    return Rotation(dims, base, scaling) if dims else None


def _heads(m: Any, where: str) -> Tuple[int, int]:
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json of {ARCHITECTURE}: {where}: {heads} heads do not divide into {kv} kv heads")
    return heads, kv


def _mask(m: Any) -> Optional[Mapping]:
    return m["mask"] if isinstance(m, Mapping) and m.get("mask") is not None else None


def _differential(m: Any, where: str) -> DifferentialMixer:
    heads, kv = _heads(m, where)
    dim, mask = _int(m, "dim", where), _mask(m)
    conv = _int(m, "conv", where) if m.get("conv") is not None else 0
    return DifferentialMixer(heads, kv, dim, _int(m, "vdim", where), _num(m, "scale", where), _num(m, "diff", where), conv,
                             _rotation(m, where, dim), _int(mask, "size", where + ".mask") if mask is not None else None)


def _windowed(m: Any, where: str) -> WindowMixer:
    heads, kv = _heads(m, where)
    dim, mask = _int(m, "dim", where), _mask(m)
    keep = _int(mask, "keep_first", where + ".mask", least=0) if mask is not None and mask.get("keep_first") is not None else 0
    return WindowMixer(heads, kv, dim, _int(m, "vdim", where), _num(m, "scale", where), _rotation(m, where, dim),
                       _int(mask, "size", where + ".mask") if mask is not None else None, keep)


def _gla(m: Any, where: str) -> GlaMixer:
    return GlaMixer(_int(m, "heads", where), _int(m, "dim", where), _int(m, "vdim", where), _num(m, "tau", where, positive=True))


_MIXERS = {"attention": _differential, "attention_2": _windowed, "gla": _gla}


def _mlp(mr: Any, where: str) -> Optional[DenseMlp]:
    if mr is None:
        return None
    if _need(mr, "kind", where) != "dense":
        raise ConfigError(f"config.json of {ARCHITECTURE}: {where}: unknown feed-forward kind {mr['kind']!r} (dense)")
    return DenseMlp(_int(mr, "ff", where), _num(mr, "limit", where, positive=True))


def _loop(lp: Any, n_layers: int) -> Optional[Loop]:
    if lp is None:
        return None
    loop = Loop(_int(lp, "start", "loop", least=0), _int(lp, "stop", "loop"), _int(lp, "times", "loop"))
    if not (loop.start < loop.stop <= n_layers):
        raise ConfigError(f"config.json of {ARCHITECTURE}: the loop over layers {loop.start} .. {loop.stop - 1} does not fit {n_layers} layers")
    return loop


@dataclass(frozen=True)
class SofopelConfig:
    architecture: str
    width: int
    vocab: int
    norm_eps: float
    embedding_scale: float
    residual_mult: float
    loop: Optional[Loop]
    layers: Tuple[SofopelLayer, ...]
    stop_token_ids: Tuple[int, ...] = ()

    # what the rest of the library asks of any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def max_position_embeddings(self) -> int:
        return NO_POSITION_LIMIT

    @property
    def eos_token_ids(self) -> Tuple[int, ...]:
        return self.stop_token_ids

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "SofopelConfig":
        width = _int(raw, "width", "the top level")
        vocab = _int(raw, "vocab", "the top level")
        layers_raw = _need(raw, "layers", "the top level")
        if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
            raise ConfigError(f"config.json of {ARCHITECTURE}: \"layers\" must be a non-empty list")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            kind, m = _need(lr, "type", where), _need(lr, "mixer", where)
            if kind not in _MIXERS:
                raise ConfigError(f"config.json of {ARCHITECTURE}: {where}: unknown layer type {kind!r} ({', '.join(_MIXERS)})")
            layers.append(SofopelLayer(kind, _MIXERS[kind](m, where), _mlp(lr.get("mlp"), where + ".mlp")))
        emb = raw.get("embedding") or {}
        stops = raw.get("eos_token_id")
        stops = () if stops is None else tuple(int(t) for t in (stops if isinstance(stops, (list, tuple)) else [stops]))
        return cls(ARCHITECTURE, width, vocab, _num(_need(raw, "norm", "the top level"), "eps", "norm"),
                   _num(emb, "scale", "embedding") if emb.get("scale") is not None else 1.0,
                   _num(raw, "residual_mult", "the top level") if raw.get("residual_mult") is not None else 1.0,
                   _loop(raw.get("loop"), len(layers)), tuple(layers), stops)


def _rotary(rot: Optional[Rotation], pairing: str) -> Optional[dict]:
    if rot is None:
        return None
    s = rot.scaling
    scaling = None if s is None else {"rope_type": "yarn", "factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
    return {"dims": rot.dims, "base": rot.base, "pairing": pairing, "scaling": scaling}


def build_sofopel_spec(cfg: SofopelConfig) -> ModelSpec:
    bare = {"tensor_names": {"weight": ""}}      # "embed", "head", "l0.norm1": the tensor is the prefix itself
    norm = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, **bare})
    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        common = {"hidden_size": cfg.width, "eps": cfg.norm_eps, "base": "mix."}
        if layer.type == "attention":
            mixer = PartSpec("differential_attention", {
                **common, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "scale": m.scale,
                "diff": m.diff, "conv": m.conv, "rotary": _rotary(m.rot, "adjacent"), "chunk": m.chunk})
        elif layer.type == "attention_2":
            mixer = PartSpec("head_normed_attention", {
                **common, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "scale": m.scale,
                "window": m.window, "keep_first": m.keep_first, "qk_norm": True, "sink": "zero", "head_gate": True,
                "rotary": _rotary(m.rot, "half")})
        else:
            mixer = PartSpec("gated_linear_attention", {**common, "heads": m.heads, "key_dim": m.dim, "v_dim": m.vdim, "tau": m.tau})
        ffn = None
        if layer.mlp is not None:
            ffn = PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": layer.mlp.ff, "activation": "clamped",
                                         "limit": layer.mlp.limit, "alpha": GATE_ALPHA,
                                         "tensor_names": {k: f"mlp.{k}" for k in ("gate", "up", "down")}})
        layers.append(LayerSpec(prefix=f"l{i}.", block="parallel_residual", mixer_norm=norm, mixer=mixer, ffn=ffn,
                                mixer_norm_prefix="norm1", block_params={"scale": cfg.residual_mult}))
    n, loop = len(layers), cfg.loop
    schedule = looped_schedule(n, loop.start, loop.stop, loop.times) if loop is not None else looped_schedule(n, n, n, 1)
    spec = ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=NO_POSITION_LIMIT,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "scale": cfg.embedding_scale, **bare}),
        layers=tuple(layers), schedule=schedule, final_norm=norm,
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied": False, **bare}),
        stop_token_ids=cfg.stop_token_ids, embedding_prefix="embed", final_norm_prefix="final.norm", head_prefix="head")
    spec.validate()
    return spec
