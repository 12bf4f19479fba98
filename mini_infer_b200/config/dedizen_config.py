"""Typed reader of a Dedizen ``config.json``.

A Dedizen model is a list of layers, each with one of three mixers and a dense feed-forward or none: a matrix memory with
exponential gates (``mlstm``), a gated linear recurrence behind a short convolution (``rglru``), or attention inside
chunks beside linear attention with fixed decays (``parallel``).  Every size and every constant that can differ between
models is read here and nowhere else.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .model_config import ConfigError

MIXER_TYPES = ("mlstm", "rglru", "parallel")
MLP_KINDS = ("dense",)


def _need(d: Mapping[str, Any], key: str, what: str):
    if key not in d:
        raise ConfigError(f"Dedizen config: {what} lacks '{key}'")
    v = d[key]
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"Dedizen config: {what} '{key}' = {v!r} has the wrong type")
    return v


def _object(d: Mapping[str, Any], key: str, what: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"Dedizen config: {what} lacks the object '{key}'")
    return v


def _whole(d: Mapping[str, Any], key: str, what: str, least: int = 1) -> int:
    v = _need(d, key, what)
    if v != int(v) or v < least:
        raise ConfigError(f"Dedizen config: {what} '{key}' = {v!r} must be a whole number of at least {least}")
    return int(v)


def _positive(d: Mapping[str, Any], key: str, what: str) -> float:
    v = float(_need(d, key, what))
    if not v > 0:
        raise ConfigError(f"Dedizen config: {what} '{key}' = {v} must be positive")
    return v


@dataclass(frozen=True)
class Mlstm:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class Rglru:
    width: int
    blocks: int
    conv: int


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
    yarn: Optional[Yarn]        # None: frequencies as they are


@dataclass(frozen=True)
class ChunkAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    chunk: int                  # 0: a query sees all earlier keys
    scale: float
    rot: Optional[Rotation]


@dataclass(frozen=True)
class FixedDecay:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class Parallel:
    left: ChunkAttention
    right: FixedDecay


@dataclass(frozen=True)
class DedizenLayer:
    mixer: Union[Mlstm, Rglru, Parallel]
    ff: Optional[int]           # None: a layer without a feed-forward


@dataclass(frozen=True)
class DedizenConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    layers: Tuple[DedizenLayer, ...]

    @classmethod
    def from_json_dict(cls, j: Mapping[str, Any]) -> "DedizenConfig":
        vocab, width = _whole(j, "vocab", "the model"), _whole(j, "width", "the model")
        eps = float(_need(_object(j, "norm", "the model"), "eps", "norm"))
        raw = j.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("Dedizen config: 'layers' must be a non-empty list")
        return cls(str(j.get("architecture", "Dedizen")), vocab, width, eps,
                   tuple(_layer(l, f"layer {i}") for i, l in enumerate(raw)))


def _layer(l: Any, what: str) -> DedizenLayer:
    if not isinstance(l, Mapping) or l.get("type") not in MIXER_TYPES:
        raise ConfigError(f"Dedizen config: {what} needs a 'type' among {MIXER_TYPES}")
    m = _object(l, "mixer", what)
    if l["type"] == "mlstm":
        mixer = Mlstm(_whole(m, "heads", what), _whole(m, "dim", what), _whole(m, "vdim", what),
                      _positive(m, "gate_cap", what))
    elif l["type"] == "rglru":
        mixer = Rglru(_whole(m, "width", what), _whole(m, "blocks", what), _whole(m, "conv", what))
        if mixer.width % mixer.blocks:
            raise ConfigError(f"Dedizen config: {what}: a width of {mixer.width} does not split into {mixer.blocks} blocks")
    else:
        mixer = Parallel(_left(_object(m, "left", what), what + " left"), _right(_object(m, "right", what), what + " right"))
    mlp, ff = l.get("mlp"), None
    if mlp is not None:
        if not isinstance(mlp, Mapping) or mlp.get("kind") not in MLP_KINDS:
            raise ConfigError(f"Dedizen config: {what} has an 'mlp' whose 'kind' is not among {MLP_KINDS}")
        ff = _whole(mlp, "ff", what + " mlp")
    return DedizenLayer(mixer, ff)


def _left(m: Mapping[str, Any], what: str) -> ChunkAttention:
    heads, kv, dim, vdim = (_whole(m, k, what) for k in ("heads", "kv_heads", "dim", "vdim"))
    if heads % kv:
        raise ConfigError(f"Dedizen config: {what}: {heads} heads over {kv} key/value heads")
    if vdim != dim:
        raise ConfigError(f"Dedizen config: {what}: the values are the keys, so 'vdim' = {vdim} must be 'dim' = {dim}")
    chunk = _whole(_object(m, "mask", what), "size", what + " mask") if m.get("mask") is not None else 0
    rot, r = None, m.get("rot")
    if r is not None and _whole(_object(m, "rot", what), "dims", what + " rot", 0):
        dims, base, yarn = _whole(r, "dims", what + " rot"), _positive(r, "base", what + " rot"), None
        if dims % 2 or dims > dim:
            raise ConfigError(f"Dedizen config: {what}: {dims} rotated dimensions of heads of {dim} (an even number)")
        if r.get("scaling") is not None:
            s = _object(r, "scaling", what + " rot")
            yarn = Yarn(*(_positive(s, k, what + " rot scaling") for k in ("factor", "original", "fast", "slow")))
            if base == 1.0:
                raise ConfigError(f"Dedizen config: {what}: a rotation of base 1 cannot be rescaled")
        rot = Rotation(dims, base, yarn)
    return ChunkAttention(heads, kv, dim, vdim, chunk, _positive(m, "scale", what), rot)


def _right(m: Mapping[str, Any], what: str) -> FixedDecay:
    heads, dim, vdim = (_whole(m, k, what) for k in ("heads", "dim", "vdim"))
    decay = m.get("decay")
    if (not isinstance(decay, (list, tuple)) or len(decay) != heads
            or not all(isinstance(v, (int, float)) and not isinstance(v, bool) and 0.0 < v <= 1.0 for v in decay)):
        raise ConfigError(f"Dedizen config: {what}: 'decay' = {decay!r} must be {heads} numbers in (0, 1]")
    return FixedDecay(heads, dim, vdim, tuple(float(v) for v in decay))
