"""Typed reader of a Gedilorn ``config.json``.

A Gedilorn model keeps several residual streams per token and is a list of layers, each with one of two forms of
attention through a latent (``latent_attention``; ``latent_attention_2``, whose output is gated) and a dense gated
feed-forward or none.  A layer may name another one whose weights it runs with (``weights_of``).  Every size and
every constant that can differ between models is read here and nowhere else.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, List, Mapping, Optional, Tuple

from .model_config import ConfigError

MIXER_TYPES = ("latent_attention", "latent_attention_2")
GATED_TYPES = ("latent_attention_2",)
MLP_KINDS = ("dense",)


def _need(d: Mapping[str, Any], key: str, what: str, kind=(int, float)):
    if key not in d:
        raise ConfigError(f"Gedilorn config: {what} lacks '{key}'")
    v = d[key]
    if isinstance(v, bool) or not isinstance(v, kind):
        raise ConfigError(f"Gedilorn config: {what} '{key}' = {v!r} has the wrong type")
    return v


def _object(d: Mapping[str, Any], key: str, what: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"Gedilorn config: {what} lacks the object '{key}'")
    return v


def _whole(d: Mapping[str, Any], key: str, what: str, least: int = 1) -> int:
    v = _need(d, key, what)
    if v != int(v) or v < least:
        raise ConfigError(f"Gedilorn config: {what} '{key}' = {v!r} must be a whole number of at least {least}")
    return int(v)


def _positive(d: Mapping[str, Any], key: str, what: str) -> float:
    v = float(_need(d, key, what))
    if not v > 0:
        raise ConfigError(f"Gedilorn config: {what} '{key}' = {v} must be positive")
    return v


@dataclass(frozen=True)
class Yarn:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class GedilornMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    base: float
    yarn: Optional[Yarn]        # None: frequencies as they are
    gated: bool


@dataclass(frozen=True)
class GedilornLayer:
    mixer: GedilornMixer
    ff: Optional[int]           # None: a layer without a feed-forward
    weights: int                # the layer whose tensors this one runs with (itself, usually)


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class GedilornConfig:
    architecture: str
    vocab: int
    width: int
    streams: int
    eps: float
    embedding_scale: float
    bigram: Optional[Bigram]
    logit_scale: float
    layers: Tuple[GedilornLayer, ...]

    @classmethod
    def from_json_dict(cls, j: Mapping[str, Any]) -> "GedilornConfig":
        vocab, width = _whole(j, "vocab", "the model"), _whole(j, "width", "the model")
        streams = _whole(j, "streams", "the model")
        eps = float(_need(_object(j, "norm", "the model"), "eps", "norm"))
        emb = _object(j, "embedding", "the model")
        bigram = None
        if emb.get("bigram") is not None:
            b = _object(emb, "bigram", "embedding")
            bigram = Bigram(_whole(b, "buckets", "bigram"), _whole(b, "mul_prev", "bigram", 0),
                            _whole(b, "mul_cur", "bigram", 0))
        raw = j.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("Gedilorn config: 'layers' must be a non-empty list")
        layers = [_layer(raw, i) for i in range(len(raw))]
        for i, l in enumerate(layers):
            own = layers[l.weights]
            if (own.mixer, own.ff) != (l.mixer, l.ff):
                raise ConfigError(f"Gedilorn config: layer {i} runs with the weights of layer {l.weights}, whose mixer "
                                  f"or feed-forward differs")
        return cls(str(j.get("architecture", "Gedilorn")), vocab, width, streams, eps,
                   float(_need(emb, "scale", "embedding")), bigram, float(_need(j, "logit_scale", "the model")),
                   tuple(layers))


def _layer(raw: List[Any], i: int) -> GedilornLayer:
    what, l = f"layer {i}", raw[i]
    if not isinstance(l, Mapping) or l.get("type") not in MIXER_TYPES:
        raise ConfigError(f"Gedilorn config: {what} needs a 'type' among {MIXER_TYPES}")
    mixer = _mixer(l["type"], _object(l, "mixer", what), what)
    mlp, ff = l.get("mlp"), None
    if mlp is not None:
        if not isinstance(mlp, Mapping) or mlp.get("kind") not in MLP_KINDS:
            raise ConfigError(f"Gedilorn config: {what} has an 'mlp' whose 'kind' is not among {MLP_KINDS}")
        ff = _whole(mlp, "ff", what + " mlp")
    # the layer that owns the tensors, through a chain of references if need be
    at, seen = i, []
    while isinstance(raw[at], Mapping) and raw[at].get("weights_of") is not None:
        seen.append(at)
        at = raw[at]["weights_of"]
        if isinstance(at, bool) or not isinstance(at, int) or not 0 <= at < len(raw) or at in seen:
            raise ConfigError(f"Gedilorn config: {what} 'weights_of' = {at!r} must name another layer")
    return GedilornLayer(mixer, ff, at)


def _mixer(kind: str, m: Mapping[str, Any], what: str) -> GedilornMixer:
    heads, dim, rot_dim, vdim, kv_rank = (_whole(m, k, what) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    rot = _object(m, "rot", what)
    if _whole(rot, "dims", what + " rot") != rot_dim or rot_dim % 2:
        raise ConfigError(f"Gedilorn config: {what}: the rotation covers {rot['dims']} dimensions, the rotated part has "
                          f"{rot_dim} (an even number)")
    base = _positive(rot, "base", what + " rot")
    yarn = None
    if rot.get("scaling") is not None:
        s = _object(rot, "scaling", what + " rot")
        yarn = Yarn(*(_positive(s, k, what + " rot scaling") for k in ("factor", "original", "fast", "slow")))
        if base == 1.0:
            raise ConfigError(f"Gedilorn config: {what}: a rotation of base 1 cannot be rescaled")
    return GedilornMixer(heads, dim, rot_dim, vdim, kv_rank, _positive(m, "scale", what), base, yarn,
                         kind in GATED_TYPES)
