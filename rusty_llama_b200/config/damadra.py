"""Typed configuration of the Damadra architecture, read from config.json.

The file lists its layers one by one; every layer names which mixer it has (`type`), the mixer's sizes and constants and
its feed-forward, so two models of the architecture may differ in everything, the order of layer kinds included.  Keys:

    architecture: "Damadra", vocab, width, norm: {eps}, embedding: {scale}, residual_mult,
    layers: [ {type: "attention", mixer: {heads, kv_heads, dim, vdim, scale, bias_max, mask: {size}}, mlp}
            | {type: "attention_2", mixer: {heads, kv_heads, dim, vdim, scale, bias_max, q_temp: {coef, every},
                                            kv_from (optional: the layer whose keys and values are read)}, mlp} ... ]
    mlp: null | {kind: "dense", ff} | {kind: "moe", router: {experts, identity, top}, expert: {ff}}

"attention" looks through a window of `mask.size` tokens, and its values are its keys before their norm (vdim = dim);
"attention_2" looks at every earlier token.  How many buckets a layer's table of distance biases has is the table's to say.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from ..errors import ConfigError
from .vezatar import _get, _int, _num

ARCHITECTURE = "Damadra"

MAX_POSITIONS = 1 << 20  # the design names no limit; the library's bookkeeping wants one


@dataclass(frozen=True)
class WindowedMixerConfig:
    heads: int
    kv_heads: int
    dim: int  # of keys and values
    scale: float
    bias_max: float
    window: int  # 0: every earlier token


@dataclass(frozen=True)
class FullMixerConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    temp_coef: float
    temp_every: int  # 0: no temperature
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    identity: int
    top: int
    ff: int


@dataclass(frozen=True)
class DamadraLayerConfig:
    type: str
    mixer: Union[WindowedMixerConfig, FullMixerConfig]
    mlp: Union[None, DenseConfig, ExpertsConfig]


@dataclass(frozen=True)
class DamadraConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    residual_mult: float
    layers: Tuple[DamadraLayerConfig, ...]
    architecture: str = ARCHITECTURE

    @classmethod
    def from_json(cls, d: Mapping[str, Any]) -> "DamadraConfig":
        layers = _get(d, "layers", "config.json")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        parsed = tuple(_layer(i, layer) for i, layer in enumerate(layers))
        for i, layer in enumerate(parsed):
            _check_source(i, layer.mixer, parsed)
        embedding = d.get("embedding")
        return cls(
            vocab=_int(d, "vocab", "config.json"),
            width=_int(d, "width", "config.json"),
            eps=_num(_get(d, "norm", "config.json"), "eps", "norm"),
            embedding_scale=1.0 if embedding is None else _num(embedding, "scale", "embedding", positive=False),
            residual_mult=_num(d, "residual_mult", "config.json", positive=False) if d.get("residual_mult") is not None else 1.0,
            layers=parsed,
        )


def _check_source(i: int, mine, parsed) -> None:
    """A layer that reads another layer's keys and values: that layer runs before it, has its own, and both agree in their shape."""
    src = getattr(mine, "kv_from", None)
    if src is None:
        return
    if not 0 <= src < i:
        raise ConfigError(f"layers[{i}].mixer.kv_from names layer {src}, which does not run before it")
    other = parsed[src].mixer
    if not isinstance(other, FullMixerConfig) or other.kv_from is not None:
        raise ConfigError(f"layers[{i}].mixer.kv_from names layer {src}, which keeps no keys and values of every token of its own")
    if (mine.kv_heads, mine.dim, mine.vdim) != (other.kv_heads, other.dim, other.vdim):
        raise ConfigError(f"layers[{i}] reads the keys and values of layer {src}, but their kv_heads, dim or vdim differ")


def _heads(m, w: str):
    heads, kv_heads = _int(m, "heads", w), _int(m, "kv_heads", w)
    if heads % kv_heads:
        raise ConfigError(f"{w}: {heads} heads are not a multiple of {kv_heads} kv_heads")
    return heads, kv_heads


def _windowed(m, w: str) -> WindowedMixerConfig:
    heads, kv_heads = _heads(m, w)
    dim, vdim = _int(m, "dim", w), _int(m, "vdim", w)
    if vdim != dim:
        raise ConfigError(f"{w}: its values are its keys, but vdim = {vdim} differs from dim = {dim}")
    if m.get("kv_from") is not None:
        raise ConfigError(f"{w}.kv_from: a layer with a window keeps keys of its own")
    mask = m.get("mask")
    return WindowedMixerConfig(heads=heads, kv_heads=kv_heads, dim=dim, scale=_num(m, "scale", w), bias_max=_num(m, "bias_max", w),
                               window=0 if mask is None else _int(mask, "size", w + ".mask"))


def _full(m, w: str) -> FullMixerConfig:
    heads, kv_heads = _heads(m, w)
    temp, coef, every = m.get("q_temp"), 0.0, 0
    if temp is not None:
        coef, every = _num(temp, "coef", w + ".q_temp", positive=False), _int(temp, "every", w + ".q_temp")
    kv_from = m.get("kv_from")
    if kv_from is not None and (isinstance(kv_from, bool) or not isinstance(kv_from, int)):
        raise ConfigError(f"{w}.kv_from must be a layer index, got {kv_from!r}")
    return FullMixerConfig(heads=heads, kv_heads=kv_heads, dim=_int(m, "dim", w), vdim=_int(m, "vdim", w), scale=_num(m, "scale", w),
                           bias_max=_num(m, "bias_max", w), temp_coef=coef, temp_every=every, kv_from=kv_from)


_MIXERS = {"attention": _windowed, "attention_2": _full}


def _mlp(mlp, where: str):
    if mlp is None:
        return None
    kind = _get(mlp, "kind", where)
    if kind == "dense":
        return DenseConfig(ff=_int(mlp, "ff", where))
    if kind == "moe":
        router = _get(mlp, "router", where)
        parsed = ExpertsConfig(
            experts=_int(router, "experts", where + ".router"), top=_int(router, "top", where + ".router"),
            identity=_int(router, "identity", where + ".router", 0) if router.get("identity") is not None else 0,
            ff=_int(_get(mlp, "expert", where), "ff", where + ".expert"),
        )
        if parsed.top > parsed.experts + parsed.identity:
            raise ConfigError(f"{where}.router: {parsed.top} of {parsed.experts} + {parsed.identity} experts per token")
        return parsed
    raise ConfigError(f"{where}.kind '{kind}' is not a feed-forward of this architecture (known: dense, moe)")


def _layer(i: int, d: Mapping[str, Any]) -> DamadraLayerConfig:
    where = f"layers[{i}]"
    kind = _get(d, "type", where)
    if kind not in _MIXERS:
        raise ConfigError(f"{where}.type '{kind}' is not a mixer of this architecture (known: {', '.join(_MIXERS)})")
    m = _get(d, "mixer", where)
    if not isinstance(m, Mapping):
        raise ConfigError(f"{where}.mixer must be an object")
    return DamadraLayerConfig(kind, _MIXERS[kind](m, where + ".mixer"), _mlp(d.get("mlp"), where + ".mlp"))
