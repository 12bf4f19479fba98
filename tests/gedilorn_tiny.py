"""Tiny Gedilorn configurations and weights for the tests.

The configurations differ from one another in every size and option: one to six residual streams, order and kinds of
layers, layers without a feed-forward, layers that run with another layer's weights (directly, through a chain, before
and after it), sizes that every kernel form takes and sizes that only the plain ones take, one head and more heads
than a tensor-core tile has rows, key, value and rotated sizes that differ, a rotated part of two numbers, YaRN ramps
that begin at zero, end at the last dimension, are a step, or are absent, bigram tables of one bucket and of more
buckets than tokens.  Weights are drawn so that scores and activations stay of order one (a model whose mixers put out
almost nothing hides their faults), and are rounded to bfloat16, so that both precision paths and the plain model read
the same numbers.
"""

from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List

import torch

PLAIN, GATED = "latent_attention", "latent_attention_2"


def _layer(kind, heads, dim, rot_dim, vdim, kv_rank, ff, base=10000.0, scaling=None, scale=None, weights_of=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    out = {"type": kind,
           "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot,
                     "scale": scale if scale is not None else (dim + rot_dim) ** -0.5},
           "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    return out if weights_of is None else dict(out, weights_of=weights_of)


def _again(layer, weights_of):
    return dict(json.loads(json.dumps(layer)), weights_of=weights_of)


def _model(vocab, width, streams, layers, eps=1e-6, scale=3.0, buckets=61, mul_prev=31, mul_cur=7, logit_scale=1.5):
    return {"architecture": "Gedilorn", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "logit_scale": logit_scale, "layers": layers}


# sizes of no kernel form but the plain ones; shared weights; a layer without a feed-forward
_A0 = _layer(GATED, 3, 8, 4, 12, 20, 80, base=100.0, scaling=(4.0, 64, 8.0, 0.5), scale=0.4)
_A1 = _layer(PLAIN, 2, 12, 6, 10, 14, None, base=1000.0, scaling=(2.0, 128, 32.0, 1.0))
CONFIG_A = _model(101, 48, 2, [_A0, _A1, _again(_A0, 0), _layer(PLAIN, 1, 20, 2, 28, 36, 56), _again(_A1, 1)], eps=1e-5)

# multiples of eight: tensor-core forms in every path; four streams; a chain of shared weights and one that stands
# before its owner
_B0 = _layer(PLAIN, 5, 24, 8, 40, 48, 96, base=50.0, scaling=(8.0, 512, 32.0, 1.0))
_B2 = _layer(GATED, 4, 40, 24, 72, 64, 64, scaling=(16.0, 256, 4.0, 0.25), scale=0.2)
CONFIG_B = _model(131, 72, 4, [_again(_B0, 1), _B0, _B2, _again(_B2, 2), _again(_B2, 3)], scale=1.0, buckets=4001,
                  mul_prev=1000003, mul_cur=131, logit_scale=0.25)

# large heads and latents, many heads, every width of the tcgen05 form's key and value tiles
CONFIG_C = _model(160, 64, 3, [
    _layer(GATED, 2, 136, 40, 128, 512, 128, scaling=(8.0, 1024, 32.0, 1.0)),
    _layer(PLAIN, 36, 16, 16, 24, 128, None, base=250.0, scaling=(3.0, 100, 1.0, 1.0)),
    _layer(GATED, 8, 32, 32, 48, 256, 64, base=5000.0),
    _layer(PLAIN, 3, 128, 64, 96, 96, 96, scaling=(40.0, 4096, 32.0, 1.0)),
    _layer(PLAIN, 16, 8, 8, 8, 64, None, scaling=(2.0, 16, 1e9, 1e-9))], buckets=1)

# one of everything that a model may happen to make equal or one
CONFIG_D = _model(64, 40, 1, [_layer(PLAIN, 1, 8, 2, 8, 8, 48, scaling=(1.0, 32, 2.0, 1.0)),
                              _layer(GATED, 1, 8, 8, 8, 8, 40, base=2.0)], eps=3e-6, scale=1.0, buckets=64, mul_prev=1,
                  mul_cur=1, logit_scale=1.0)

# more streams than the register form holds, a width that is no multiple of four
CONFIG_E = _model(90, 54, 6, [_layer(GATED, 2, 16, 8, 16, 32, 64), _layer(PLAIN, 6, 8, 4, 8, 16, 32, scaling=(4.0, 64, 4.0, 1.0))],
                  buckets=17, mul_prev=0, mul_cur=5)

CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D, "E": CONFIG_E}


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """``name -> bfloat16 tensor`` for every tensor the configuration implies (names built here from the
    configuration alone, so the engine's own manifest is checked against an independent one)."""
    g = torch.Generator().manual_seed(seed)
    W, S = cfg["width"], cfg["streams"]

    def rnd(*shape, std=1.0):
        return torch.randn(*shape, generator=g) * std

    def lin(out, inn, gain=1.0):
        return rnd(out, inn, std=gain / math.sqrt(inn))

    def gain(n):
        return 1.0 + rnd(n, std=0.2)

    def streams(p):
        w[p + "in"], w[p + "out"] = 1.0 / S + rnd(S, std=0.3), 0.8 + rnd(S, std=0.3)
        w[p + "mix"] = 0.8 * torch.eye(S) + rnd(S, S, std=0.15)

    w: Dict[str, torch.Tensor] = {"embed": rnd(cfg["vocab"], W), "embed.norm": gain(W), "head": lin(cfg["vocab"], W, 2.0),
                                  "final.norm": gain(W)}
    if cfg["embedding"].get("bigram"):
        w["bigram"] = rnd(cfg["embedding"]["bigram"]["buckets"] + 1, W, std=2.0)
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", L["mixer"]
        H, d, r, e, c = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        w[p + "norm1"] = gain(W)
        streams(p + "hc1.")
        q = p + "mix."
        w[q + "q"] = lin(H * (d + r), W, 1.5)
        w[q + "dkv"], w[q + "dkv.norm"] = lin(c + r, W), gain(c)
        w[q + "uk"], w[q + "uv"] = lin(H * d, c, 1.2), lin(H * e, c, 1.2)
        if L["type"] == GATED:
            w[q + "g"] = lin(H * e, W, 2.0)
        w[q + "o"] = lin(W, H * e, 1.5)
        if L.get("mlp") is not None:
            ff = L["mlp"]["ff"]
            w[p + "norm2"] = gain(W)
            streams(p + "hc2.")
            q = p + "mlp."
            w[q + "gate"], w[q + "up"], w[q + "down"] = lin(ff, W), lin(ff, W), lin(W, ff, 1.5)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def write_folder(folder: str, cfg: dict, weights: Dict[str, torch.Tensor]) -> str:
    """``config.json`` and ``model.safetensors`` (8-byte length, JSON header, data) written by hand."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, off = {}, [], 0
    for name, t in weights.items():
        raw = t.contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    hj = json.dumps(header).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)))
        f.write(hj)
        for b in blobs:
            f.write(b)
    return folder


def random_requests(cfg: dict, lengths: List[int], seed: int) -> Dict[str, List[int]]:
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}


def random_config(seed: int) -> dict:
    """A configuration drawn at random: sizes, order and kinds of layers, shared weights, constants."""
    import random
    r = random.Random(seed)
    step = r.choice([1, 4, 8, 8, 16])            # what head and latent sizes are multiples of

    def size(lo, hi):
        return step * r.randint(max(1, lo // step), max(1, hi // step))
    layers = []
    for i in range(r.randint(2, 5)):
        owners = [j for j, l in enumerate(layers) if "weights_of" not in l]
        if owners and r.random() < 0.3:
            j = r.choice(owners)
            layers.append(_again(layers[j], j))
            continue
        scaling = None if r.random() < 0.2 else (r.choice([2.0, 8.0, 32.0]), r.choice([64, 512, 4096]),
                                                 r.choice([4.0, 32.0]), r.choice([0.25, 1.0]))
        layers.append(_layer(r.choice([PLAIN, GATED]), r.choice([1, 2, 3, 4, 7, 8, 12, 16]), size(8, 72),
                             2 * r.randint(1, 20) if step < 8 else 8 * r.randint(1, 6), size(8, 96), size(16, 160),
                             r.choice([None, 40, 64, 96]), base=r.choice([30.0, 10000.0, 250000.0]), scaling=scaling))
    return _model(r.randint(50, 200), r.choice([40, 64, 66, 96]), r.randint(1, 5), layers, eps=r.choice([1e-5, 1e-6]),
                  scale=r.choice([0.5, 4.0, 16.0]), buckets=r.randint(2, 300), mul_prev=r.randint(1, 5000),
                  mul_cur=r.randint(1, 5000), logit_scale=r.choice([0.3, 1.0, 2.5]))
