"""``Dedizen`` described as an arrangement of parts.

A pre-norm decoder (``prenorm_residual``) of three kinds of layers:

* ``mlstm``     a matrix memory per head with exponential input gates and logistic forget gates, kept bounded by a running
                maximum and read out through a normaliser (``matrix_lstm``)
* ``rglru``     a gated linear recurrence per channel behind a short convolution, times a second branch (``gated_lru``)
* ``parallel``  two mixers that read the same input; each output is normalised over the model width and half of each is
                added.  Left: grouped-query attention inside chunks of positions whose values are the keys as projected,
                with YaRN-scaled rotation of neighbouring dimensions, queries and keys brought to unit root mean square
                after it, a learned sink per head and a gate per head (``head_mix_attention``).  Right: linear attention
                with a fixed decay per head (``fixed_decay_attention``)

The feed-forward is dense with a squared rectifier (``squared_relu_mlp``), or none.  The output head is the embedding
table.  Nothing here computes: the function turns ``config.json`` into a :class:`ModelSpec`.
"""

from __future__ import annotations

from typing import Any, Dict

from ..config.dedizen_config import ChunkAttention, DedizenConfig, FixedDecay, Mlstm, Rglru
from ..config.registry import register_architecture
from ..config.spec import LayerPart, LayerSpec, ModelSpec, PartSpec, ScheduleEntry

PARALLEL_SCALE = 0.5        # of each of the two outputs


def _norm(c: DedizenConfig, tensor: str) -> PartSpec:
    return PartSpec("rmsnorm", {"size": c.width, "eps": c.eps, "tensor": tensor})


def _mlstm(c: DedizenConfig, m: Mlstm) -> PartSpec:
    return PartSpec("matrix_lstm", {"hidden_size": c.width, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim,
                                    "gate_cap": m.gate_cap, "eps": c.eps})


def _rglru(c: DedizenConfig, m: Rglru) -> PartSpec:
    return PartSpec("gated_lru", {"hidden_size": c.width, "width": m.width, "blocks": m.blocks, "conv": m.conv})


def _attention(c: DedizenConfig, m: ChunkAttention) -> PartSpec:
    position = PartSpec("none")
    if m.rot is not None:
        rot = {"head_dim": m.dim, "rot_dim": m.rot.dims, "theta": m.rot.base, "pairing": "neighbours"}
        y = m.rot.yarn
        if y is not None:
            rot.update(factor=y.factor, original=y.original, fast=y.fast, slow=y.slow)
        position = PartSpec("rope" if y is None else "rope_yarn", rot)
    return PartSpec("head_mix_attention", {
        "hidden_size": c.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
        "chunk": m.chunk, "scale": m.scale, "position": position, "bias": True, "values": "keys",
        "qk_norm": {"eps": c.eps, "after_rotation": True, "gain": False}, "sink": "learned", "output_gate": "heads"})


def _fixed_decay(c: DedizenConfig, m: FixedDecay) -> PartSpec:
    return PartSpec("fixed_decay_attention", {"hidden_size": c.width, "num_heads": m.heads, "head_dim": m.dim,
                                              "value_dim": m.vdim, "decay": list(m.decay), "eps": c.eps})


def build_dedizen(config_json: Dict[str, Any]) -> ModelSpec:
    c = DedizenConfig.from_json_dict(config_json)
    layers, unused = [], []
    for i, l in enumerate(c.layers):
        parts = {"mixer_norm": LayerPart("norm", _norm(c, "norm1"), "")}
        block = {"feed_forward": l.ff is not None}
        if isinstance(l.mixer, Mlstm):
            parts["mixer"] = LayerPart("mixer", _mlstm(c, l.mixer), "mix.")
        elif isinstance(l.mixer, Rglru):
            parts["mixer"] = LayerPart("mixer", _rglru(c, l.mixer), "mix.")
        else:
            parts["mixer"] = LayerPart("mixer", _attention(c, l.mixer.left), "mix.left.")
            parts["mixer_b"] = LayerPart("mixer", _fixed_decay(c, l.mixer.right), "mix.right.")
            parts["mixer_out_norm"] = LayerPart("norm", _norm(c, "out"), "mix.left.")
            parts["mixer_b_out_norm"] = LayerPart("norm", _norm(c, "out"), "mix.right.")
            block.update(second_mixer=True, mixer_scale=PARALLEL_SCALE, second_mixer_scale=PARALLEL_SCALE)
        if l.ff is not None:
            parts["feed_forward_norm"] = LayerPart("norm", _norm(c, "norm2"), "")
            parts["feed_forward"] = LayerPart("feed_forward", PartSpec("squared_relu_mlp", {
                "hidden_size": c.width, "intermediate_size": l.ff, "up": "up", "down": "down"}), "mlp.")
        else:
            unused.append(f"l{i}.norm2")        # a layer without a feed-forward may still carry its norm
        layers.append(LayerSpec(f"l{i}", PartSpec("prenorm_residual", block), parts))
    return ModelSpec(
        architecture=c.architecture, hidden_size=c.width, vocab_size=c.vocab, max_context=1 << 30,
        embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": c.width, "tensor": "embed"}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=_norm(c, "final.norm"),
        lm_head=PartSpec("linear", {"vocab_size": c.vocab, "hidden_size": c.width, "tied_to": "embed"}),
        embedding_prefix="", final_norm_prefix="", lm_head_prefix="", unused_tensors=tuple(unused))


register_architecture("Dedizen", build_dedizen,
                      "Dedizen decoder (matrix memories with exponential gates, gated linear recurrences behind short "
                      "convolutions, attention inside chunks with values that are the keys and a learned sink beside "
                      "linear attention with fixed decays; dense feed-forward with a squared rectifier)")
