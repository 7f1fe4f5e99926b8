"""Typed configuration of the Vavupel decoder, read from config.json, and the layers it is made of.

A Vavupel model adds a table of token pairs to its token embedding (`embedding.scale`, `embedding.bigram` = {`buckets`,
`mul_prev`, `mul_cur`}), norms the sum, and runs a list of layers, some of them several times over: with `loop` = {`start`,
`stop`, `times`} the layers start .. stop - 1 run `times` times in a row on the same weights (each pass with a cache or state of
its own), and before every pass the stream is replaced by a product of itself and the embedding output side by side.  Every
norm across the width is an element-wise tanh (its alpha, weight and bias are tensors), one before and one after each sublayer.
`layers[i].type` names the mixer, `layers[i].mixer` gives its sizes:

* "latent_attention": attention in a sliding window (`mask.size`) whose keys and values come out of one cached latent per token
  (`kv_rank`), `dim` unrotated and `rot_dim` rotated numbers per head (neighbouring pairs turn, `rot.base`), `scale`, a learned
  sink and one sigmoid gate per head;
* "retention": linear attention with a constant `decay` per head, rotated queries and keys (pairs half of `rot.dims` apart).

The feed-forward (`mlp.kind` "dense") is W_down relu(W_up h)^2; `mlp` null: none.  The head is a matrix of its own, its logits
capped by `logit_softcap`.  Nothing about a model lives in code: sizes, counts, constants and the order of layers come from
config.json.

Tensors: "embed", "bigram", "embed.norm", "loop.in", "l<i>.norm1", "l<i>.norm1b", "l<i>.norm2", "l<i>.norm2b", "l<i>.mix.*",
"l<i>.mlp.{up,down}", "final.norm", "head"; a norm's tensors are its name, and that with ".b" and ".alpha".
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..parts.spec import ExtraPart, LayerSpec, ModelSpec, PartSpec, looped_schedule
from .errors import ConfigError

ARCHITECTURE = "Vavupel"
# rotary angles are formed from the position itself: no length the design was trained for is written anywhere
NO_POSITION_LIMIT = 1 << 20


def _need(d: Any, key: str, where: str):
    if not isinstance(d, Mapping) or key not in d or d[key] is None:
        raise ConfigError(f"config.json of {ARCHITECTURE}: missing key \"{key}\" in {where}")
    return d[key]


def _int(d: Any, key: str, where: str, least: int = 1) -> int:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or int(v) != v or int(v) < least:
        raise ConfigError(f"config.json of {ARCHITECTURE}: \"{key}\" in {where} must be an integer >= {least}, got {v!r}")
    return int(v)


def _num(d: Any, key: str, where: str) -> float:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json of {ARCHITECTURE}: \"{key}\" in {where} must be a number, got {v!r}")
    return float(v)


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float


@dataclass(frozen=True)
class PairTable:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Optional[Rotation]
    window: Optional[int]


@dataclass(frozen=True)
class RetentionMixer:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[Rotation]


@dataclass(frozen=True)
class DenseMlp:
    ff: int


@dataclass(frozen=True)
class VavupelLayer:
    type: str
    mixer: Any
    mlp: Optional[DenseMlp]


def _rotation(m: Any, where: str, most: int) -> Optional[Rotation]:
    if not isinstance(m, Mapping) or m.get("rot") is None:
        return None
    r = m["rot"]
    dims = _int(r, "dims", where + ".rot", least=0)
    if dims % 2 or dims > most:
        raise ConfigError(f"config.json of {ARCHITECTURE}: {where}.rot: {dims} rotated numbers must be even and at most {most}")
    base = _num(r, "base", where + ".rot")
    if base <= 0:
        raise ConfigError(f"config.json of {ARCHITECTURE}: {where}.rot: base must be positive, got {base}")
    return Rotation(dims, base) if dims else None


def _latent(m: Any, where: str) -> LatentMixer:
    rot_dim = _int(m, "rot_dim", where, least=0)
    window = _int(m["mask"], "size", where + ".mask") if isinstance(m, Mapping) and m.get("mask") is not None else None
    return LatentMixer(_int(m, "heads", where), _int(m, "dim", where), rot_dim, _int(m, "vdim", where), _int(m, "kv_rank", where),
                       _num(m, "scale", where), _rotation(m, where, rot_dim), window)


def _retention(m: Any, where: str) -> RetentionMixer:
    heads, dim = _int(m, "heads", where), _int(m, "dim", where)
    decay = _need(m, "decay", where)
    if not isinstance(decay, (list, tuple)) or len(decay) != heads or any(isinstance(g, bool) or not isinstance(g, (int, float)) for g in decay):
        raise ConfigError(f"config.json of {ARCHITECTURE}: {where}: \"decay\" must list one number per head ({heads})")
    return RetentionMixer(heads, dim, _int(m, "vdim", where), tuple(float(g) for g in decay), _rotation(m, where, dim))


_MIXERS = {"latent_attention": _latent, "retention": _retention}


def _mlp(mr: Any, where: str) -> Optional[DenseMlp]:
    if mr is None:
        return None
    if _need(mr, "kind", where) != "dense":
        raise ConfigError(f"config.json of {ARCHITECTURE}: {where}: unknown feed-forward kind {mr['kind']!r} (dense)")
    return DenseMlp(_int(mr, "ff", where))


def _loop(lp: Any, n_layers: int) -> Optional[Loop]:
    if lp is None:
        return None
    loop = Loop(_int(lp, "start", "loop", least=0), _int(lp, "stop", "loop"), _int(lp, "times", "loop"))
    if not (loop.start < loop.stop <= n_layers):
        raise ConfigError(f"config.json of {ARCHITECTURE}: the loop over layers {loop.start} .. {loop.stop - 1} does not fit {n_layers} layers")
    return loop


@dataclass(frozen=True)
class VavupelConfig:
    architecture: str
    width: int
    vocab: int
    norm_eps: float
    embedding_scale: float
    pairs: Optional[PairTable]
    loop: Optional[Loop]
    logit_softcap: Optional[float]
    layers: Tuple[VavupelLayer, ...]
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
    def from_dict(cls, raw: Mapping[str, Any]) -> "VavupelConfig":
        width = _int(raw, "width", "the top level")
        vocab = _int(raw, "vocab", "the top level")
        emb = raw.get("embedding") or {}
        pairs = None
        if emb.get("bigram") is not None:
            b, where = emb["bigram"], "embedding.bigram"
            pairs = PairTable(_int(b, "buckets", where), _int(b, "mul_prev", where, least=0), _int(b, "mul_cur", where, least=0))
        layers_raw = _need(raw, "layers", "the top level")
        if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
            raise ConfigError(f"config.json of {ARCHITECTURE}: \"layers\" must be a non-empty list")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            kind, m = _need(lr, "type", where), _need(lr, "mixer", where)
            if kind not in _MIXERS:
                raise ConfigError(f"config.json of {ARCHITECTURE}: {where}: unknown layer type {kind!r} ({', '.join(_MIXERS)})")
            layers.append(VavupelLayer(kind, _MIXERS[kind](m, where), _mlp(lr.get("mlp"), where + ".mlp")))
        cap = _num(raw, "logit_softcap", "the top level") if raw.get("logit_softcap") is not None else None
        if cap is not None and not cap > 0:
            raise ConfigError(f"config.json of {ARCHITECTURE}: logit_softcap must be positive, got {cap}")
        stops = raw.get("eos_token_id")
        stops = () if stops is None else tuple(int(t) for t in (stops if isinstance(stops, (list, tuple)) else [stops]))
        return cls(ARCHITECTURE, width, vocab, _num(_need(raw, "norm", "the top level"), "eps", "norm"),
                   _num(emb, "scale", "embedding") if emb.get("scale") is not None else 1.0, pairs,
                   _loop(raw.get("loop"), len(layers)), cap, tuple(layers), stops)


def build_vavupel_spec(cfg: VavupelConfig) -> ModelSpec:
    bare = {"tensor_names": {"weight": ""}}      # "embed", "head", "loop.in": the tensor is the prefix itself
    norm = PartSpec("dynamic_tanh", {"size": cfg.width, "tensor_names": {"weight": "", "bias": ".b", "alpha": ".alpha"}})
    layers, ignorable = [], []
    for i, layer in enumerate(cfg.layers):
        m, p = layer.mixer, f"l{i}."
        rotary = lambda head, pairing: None if m.rot is None else PartSpec(
            "rotary", {"head_dim": head, "rotary_dim": m.rot.dims, "theta": m.rot.base, "pairing": pairing})
        if layer.type == "latent_attention":
            mixer = PartSpec("latent_attention", {
                "hidden_size": cfg.width, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_head_dim": m.vdim,
                "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps, "position": rotary(m.rot_dim, "adjacent"),
                "window": m.window, "sink": True, "out_gate": "head_sigmoid"})
        else:
            mixer = PartSpec("retention", {
                "hidden_size": cfg.width, "heads": m.heads, "key_dim": m.dim, "v_dim": m.vdim, "decay": m.decay, "eps": cfg.norm_eps,
                "position": rotary(m.dim, "half"), "base": "mix."})
        extra = [ExtraPart("mixer_post", "norm", norm, "norm1b")]
        ffn = None
        if layer.mlp is not None:
            ffn = PartSpec("mlp", {"hidden_size": cfg.width, "intermediate_size": layer.mlp.ff, "activation": "relu2", "bias": False})
            extra.append(ExtraPart("ffn_post", "norm", norm, "norm2b"))
        else:
            ignorable += [f"{p}{n}{t}" for n in ("norm2", "norm2b") for t in ("", ".b", ".alpha")]
        layers.append(LayerSpec(prefix=p, block="sandwich_residual", mixer_norm=norm, mixer=mixer, ffn_norm=norm if ffn is not None else None,
                                ffn=ffn, mixer_norm_prefix="norm1", ffn_norm_prefix="norm2", extra=tuple(extra)))
    n = len(layers)
    loop = cfg.loop
    schedule = looped_schedule(n, loop.start, loop.stop, loop.times, inject=True) if loop is not None else looped_schedule(n, n, n, 1)
    table = {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "scale": cfg.embedding_scale, **bare}
    if cfg.pairs is not None:
        b = cfg.pairs
        embedding = PartSpec("token_pair_embedding", {**table, "pairs": "bigram", "buckets": b.buckets, "mul_prev": b.mul_prev, "mul_cur": b.mul_cur})
    else:
        embedding = PartSpec("token_embedding", table)
    spec = ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=NO_POSITION_LIMIT,
        embedding=embedding, layers=tuple(layers), schedule=schedule, final_norm=norm,
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied": False, "softcap": cfg.logit_softcap, **bare}),
        stop_token_ids=cfg.stop_token_ids, embedding_prefix="embed", final_norm_prefix="final.norm", head_prefix="head",
        ignorable_tensors=tuple(ignorable), embedding_norm=norm, embedding_norm_prefix="embed.norm",
        injection=PartSpec("input_injection", {"hidden_size": cfg.width, **bare}) if loop is not None else None,
        injection_prefix="loop.in")
    spec.validate()
    return spec
