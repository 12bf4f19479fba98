"""``Gedilorn`` described as an arrangement of parts.

A decoder of several parallel residual streams that every sublayer reads and writes through small matrices
(``hyper_connections``).  Its embedding adds to a token's scaled row the row of a second table that a hash of the
token and the one before it picks, and brings the sum to unit root mean square (``token_embedding`` with ``bigram``).
Each layer has attention through a latent over all earlier tokens, rotated by YaRN-scaled angles, with or without a
gate on its output (``latent_attention``), and a dense feed-forward with rectified gates (``gated_mlp``) or none.
A layer may run with another layer's weights and a cache of its own: the schedule names that layer twice.

Nothing here computes: the function turns ``config.json`` into a :class:`ModelSpec`.
"""

from __future__ import annotations

from typing import Any, Dict

from ..config.gedilorn_config import GedilornConfig, GedilornMixer
from ..config.registry import register_architecture
from ..config.spec import LayerPart, LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _norm(c: GedilornConfig, tensor: str, gain: float = 1.0) -> PartSpec:
    return PartSpec("rmsnorm", {"size": c.width, "eps": c.eps, "tensor": tensor, "gain": gain})


def _mixer(c: GedilornConfig, m: GedilornMixer) -> PartSpec:
    rot = {"head_dim": m.rot_dim, "theta": m.base, "pairing": "neighbours"}
    if m.yarn is not None:
        rot.update(factor=m.yarn.factor, original=m.yarn.original, fast=m.yarn.fast, slow=m.yarn.slow)
    return PartSpec("latent_attention", {
        "hidden_size": c.width, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim,
        "kv_rank": m.kv_rank, "q_rank": 0, "window": 0, "scale": m.scale, "eps": c.eps, "output_gate": m.gated,
        "position": PartSpec("rope_yarn" if m.yarn is not None else "rope", rot)})


def build_gedilorn(config_json: Dict[str, Any]) -> ModelSpec:
    c = GedilornConfig.from_json_dict(config_json)
    layers, index, unused = [], {}, []
    for i, l in enumerate(c.layers):
        if l.weights != i:
            continue
        parts = {"mixer_norm": LayerPart("norm", _norm(c, "norm1")), "mixer": LayerPart("mixer", _mixer(c, l.mixer), "mix.")}
        block = {"streams": c.streams, "feed_forward": l.ff is not None, "mixer_streams": "hc1."}
        if l.ff is not None:
            block["feed_forward_streams"] = "hc2."
            parts["feed_forward_norm"] = LayerPart("norm", _norm(c, "norm2"))
            parts["feed_forward"] = LayerPart("feed_forward", PartSpec("gated_mlp", {
                "hidden_size": c.width, "intermediate_size": l.ff, "activation": "relu",
                "gate": "gate", "up": "up", "down": "down"}), "mlp.")
        else:
            # a layer without a feed-forward may still carry the tensors around it
            unused += [f"l{i}.norm2"] + [f"l{i}.hc2.{n}" for n in ("in", "out", "mix")]
        index[i] = len(layers)
        layers.append(LayerSpec(f"l{i}", PartSpec("hyper_connections", block), parts))
    embedding = {"vocab_size": c.vocab, "hidden_size": c.width, "tensor": "embed", "scale": c.embedding_scale,
                 "norm": _norm(c, "embed.norm"), "streams": c.streams}
    if c.bigram is not None:
        embedding["bigram"] = {"tensor": "bigram", "buckets": c.bigram.buckets, "mul_prev": c.bigram.mul_prev,
                               "mul_cur": c.bigram.mul_cur}
    return ModelSpec(
        architecture=c.architecture, hidden_size=c.width, vocab_size=c.vocab, max_context=1 << 30,
        embedding=PartSpec("token_embedding", embedding),
        layers=tuple(layers),
        # every run of a layer owns a cache, also where two runs share their weights
        schedule=tuple(ScheduleEntry(index[l.weights]) for l in c.layers),
        # the head is linear: the factor on the logits is taken into the last norm's weight
        final_norm=_norm(c, "final.norm", gain=c.logit_scale),
        lm_head=PartSpec("linear", {"vocab_size": c.vocab, "hidden_size": c.width, "tied_to": None, "tensor": "head"}),
        embedding_prefix="", final_norm_prefix="", lm_head_prefix="", unused_tensors=tuple(unused))


register_architecture("Gedilorn", build_gedilorn,
                      "Gedilorn decoder (parallel residual streams with hyper-connections, hashed bigram embedding, "
                      "attention through latents with YaRN-scaled rotation and an optional output gate, dense "
                      "feed-forward with rectified gates, layers that share weights)")
