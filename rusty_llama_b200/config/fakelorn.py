"""Typed configuration of the Fakelorn architecture, read from config.json.

The file lists its layers one by one; every layer names which mixer it has (`type`), the mixer's sizes and constants and
its feed-forward, so two models of the architecture may differ in everything, the order of layer kinds included.  Keys:

    architecture: "Fakelorn", vocab, width, norm: {eps, groups}, logit_scale, logit_softcap (null or absent: no cap),
    layers: [ {type: "attention", mixer: {heads, kv_heads, dim, vdim, scale, diff, mask: {size}}, mlp}
            | {type: "mamba2", mixer: {heads, vdim, state, groups, conv, norm_groups}, mlp}
            | {type: "latent_attention", mixer: {heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot: {base, dims},
                                                 kv_from (optional: the layer whose cache is read)}, mlp} ... ]
    mlp: null | {kind: "dense", ff} | {kind: "moe", router: {experts, top}, expert: {ff}, shared: {ff} or null}

What else a layer has (the gates on its two results, the latents of its queries, the output gate) belongs to the design.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from ..errors import ConfigError
from .vezatar import _get, _int, _num

ARCHITECTURE = "Fakelorn"

MAX_POSITIONS = 1 << 20  # the design names no limit; the library's bookkeeping wants one


@dataclass(frozen=True)
class AttentionMixerConfig:
    heads: int
    kv_heads: int
    dim: int  # of one of a head's two maps
    vdim: int
    scale: float
    diff: float
    window: int  # 0: every earlier token


@dataclass(frozen=True)
class Mamba2MixerConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class LatentMixerConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    top: int
    ff: int
    shared_ff: int = 0  # 0: no shared expert


@dataclass(frozen=True)
class FakelornLayerConfig:
    type: str
    mixer: Union[AttentionMixerConfig, Mamba2MixerConfig, LatentMixerConfig]
    mlp: Union[None, DenseConfig, ExpertsConfig]


@dataclass(frozen=True)
class FakelornConfig:
    vocab: int
    width: int
    eps: float
    norm_groups: int
    logit_scale: float
    logit_softcap: float  # 0: no cap
    layers: Tuple[FakelornLayerConfig, ...]
    architecture: str = ARCHITECTURE

    @classmethod
    def from_json(cls, d: Mapping[str, Any]) -> "FakelornConfig":
        layers = _get(d, "layers", "config.json")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        parsed = tuple(_layer(i, layer) for i, layer in enumerate(layers))
        for i, layer in enumerate(parsed):
            _check_source(i, layer.mixer, parsed)
        width = _int(d, "width", "config.json")
        norm = _get(d, "norm", "config.json")
        groups = _int(norm, "groups", "norm") if norm.get("groups") is not None else 1
        if width % groups:
            raise ConfigError(f"norm.groups = {groups} does not divide the width {width}")
        cap = _num(d, "logit_softcap", "config.json", positive=False) if d.get("logit_softcap") is not None else 0.0
        if cap < 0:
            raise ConfigError(f"logit_softcap = {cap} must not be negative (0: no cap)")
        return cls(
            vocab=_int(d, "vocab", "config.json"),
            width=width,
            eps=_num(norm, "eps", "norm"),
            norm_groups=groups,
            logit_scale=_num(d, "logit_scale", "config.json", positive=False) if d.get("logit_scale") is not None else 1.0,
            logit_softcap=cap,
            layers=parsed,
        )


def _check_source(i: int, mine, parsed) -> None:
    """A layer that reads another layer's latents: that layer runs before it, has latents of its own, and both agree in their shape and rotation."""
    src = getattr(mine, "kv_from", None)
    if src is None:
        return
    if not 0 <= src < i:
        raise ConfigError(f"layers[{i}].mixer.kv_from names layer {src}, which does not run before it")
    other = parsed[src].mixer
    if not isinstance(other, LatentMixerConfig) or other.kv_from is not None:
        raise ConfigError(f"layers[{i}].mixer.kv_from names layer {src}, which keeps no latents of its own")
    if (mine.kv_rank, mine.rot_dim, mine.rot_base, mine.rot_dims) != (other.kv_rank, other.rot_dim, other.rot_base, other.rot_dims):
        raise ConfigError(f"layers[{i}] reads the latents of layer {src}, but their kv_rank, rot_dim or rotation differ")


def _attention(m, w: str) -> AttentionMixerConfig:
    heads, kv_heads = _int(m, "heads", w), _int(m, "kv_heads", w)
    if heads % kv_heads:
        raise ConfigError(f"{w}: {heads} heads are not a multiple of {kv_heads} kv_heads")
    mask = m.get("mask")
    return AttentionMixerConfig(
        heads=heads, kv_heads=kv_heads, dim=_int(m, "dim", w), vdim=_int(m, "vdim", w), scale=_num(m, "scale", w),
        diff=_num(m, "diff", w, positive=False), window=0 if mask is None else _int(mask, "size", w + ".mask"),
    )


def _mamba2(m, w: str) -> Mamba2MixerConfig:
    c = Mamba2MixerConfig(heads=_int(m, "heads", w), vdim=_int(m, "vdim", w), state=_int(m, "state", w), groups=_int(m, "groups", w),
                          conv=_int(m, "conv", w), norm_groups=_int(m, "norm_groups", w))
    if c.heads % c.groups:
        raise ConfigError(f"{w}: {c.heads} heads are not a multiple of {c.groups} groups")
    if (c.heads * c.vdim) % c.norm_groups:
        raise ConfigError(f"{w}.norm_groups = {c.norm_groups} does not divide heads * vdim = {c.heads * c.vdim}")
    return c


def _latent(m, w: str) -> LatentMixerConfig:
    rot_dim = _int(m, "rot_dim", w, 0)
    rot = m.get("rot")
    base, dims = 10000.0, 0
    if rot is not None:
        base, dims = _num(rot, "base", w + ".rot"), _int(rot, "dims", w + ".rot", 0)
    if dims > rot_dim or dims % 2:
        raise ConfigError(f"{w}.rot.dims = {dims} must be even and at most rot_dim = {rot_dim}")
    kv_from = m.get("kv_from")
    if kv_from is not None and (isinstance(kv_from, bool) or not isinstance(kv_from, int)):
        raise ConfigError(f"{w}.kv_from must be a layer index, got {kv_from!r}")
    return LatentMixerConfig(
        heads=_int(m, "heads", w), dim=_int(m, "dim", w, 0), rot_dim=rot_dim, vdim=_int(m, "vdim", w), q_rank=_int(m, "q_rank", w),
        kv_rank=_int(m, "kv_rank", w), scale=_num(m, "scale", w), rot_base=base, rot_dims=dims, kv_from=kv_from,
    )


_MIXERS = {"attention": _attention, "mamba2": _mamba2, "latent_attention": _latent}


def _mlp(mlp, where: str):
    if mlp is None:
        return None
    kind = _get(mlp, "kind", where)
    if kind == "dense":
        return DenseConfig(ff=_int(mlp, "ff", where))
    if kind == "moe":
        router, shared = _get(mlp, "router", where), mlp.get("shared")
        parsed = ExpertsConfig(
            experts=_int(router, "experts", where + ".router"), top=_int(router, "top", where + ".router"),
            ff=_int(_get(mlp, "expert", where), "ff", where + ".expert"),
            shared_ff=_int(shared, "ff", where + ".shared") if shared is not None else 0,
        )
        if parsed.top > parsed.experts:
            raise ConfigError(f"{where}.router: {parsed.top} of {parsed.experts} experts per token")
        return parsed
    raise ConfigError(f"{where}.kind '{kind}' is not a feed-forward of this architecture (known: dense, moe)")


def _layer(i: int, d: Mapping[str, Any]) -> FakelornLayerConfig:
    where = f"layers[{i}]"
    kind = _get(d, "type", where)
    if kind not in _MIXERS:
        raise ConfigError(f"{where}.type '{kind}' is not a mixer of this architecture (known: {', '.join(_MIXERS)})")
    m = _get(d, "mixer", where)
    if not isinstance(m, Mapping):
        raise ConfigError(f"{where}.mixer must be an object")
    return FakelornLayerConfig(kind, _MIXERS[kind](m, where + ".mixer"), _mlp(d.get("mlp"), where + ".mlp"))
