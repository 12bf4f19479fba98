"""Tiny Dedizen configurations and weights for the tests.

The configurations differ from one another in every size and option: number and order of layers, layers without a
feed-forward (also behind a pair of mixers, and last), matrix memories with keys longer and shorter than values and with
sizes that no tile divides, parts of the recurrence of one, three and more channels, one part or several, convolutions of
one to five taps, heads that share a key/value head or do not, chunks of 1, 3, 10 and more positions, rotation of a whole
head, of part of it, of none, with and without rescaled frequencies, decays near 0 and of exactly 1.  Weights are drawn so
that scores, gates and decays stay away from their saturated ends and are rounded to bfloat16, so that both precision
paths and the plain model read the same numbers.
"""

from __future__ import annotations

import math
from typing import Dict

import torch

from nipapel_tiny import random_requests, write_folder  # noqa: F401  (container writer and request maker)


def _ff(n):
    return None if n is None else {"kind": "dense", "ff": n}


def _mlstm(heads, dim, vdim, cap, ff):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": _ff(ff)}


def _rglru(width, blocks, conv, ff):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": _ff(ff)}


def _rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def _parallel(heads, kv, dim, chunk, scale, rot, decay, rdim, rvdim, ff):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "mask": {"size": chunk}, "scale": scale}
    if rot is not None:
        left["rot"] = rot
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": len(decay), "dim": rdim, "vdim": rvdim,
                                                                  "decay": list(decay)}}, "mlp": _ff(ff)}


CONFIG_A = {
    "architecture": "Dedizen", "vocab": 101, "width": 48, "norm": {"eps": 1e-5},
    "layers": [
        _parallel(4, 2, 12, 10, 0.5, _rot(8, 500.0, (4.0, 64, 8.0, 1.0)), [0.7, 0.95, 0.99], 10, 6, 40),
        _mlstm(3, 10, 14, 6.0, 72),
        _rglru(30, 3, 3, None),
        _parallel(5, 1, 16, 3, 0.4, _rot(16, 10000.0, (2.5, 40, 6.0, 0.5)), [0.5], 12, 20, None),
        _rglru(36, 1, 1, 24),
        _mlstm(1, 24, 8, 15.0, None),
    ],
}

CONFIG_B = {
    "architecture": "Dedizen", "vocab": 131, "width": 72, "norm": {"eps": 1e-6},
    "layers": [
        _rglru(44, 44, 5, 56),
        _mlstm(4, 6, 10, 3.0, None),
        _mlstm(2, 33, 17, 10.0, 20),
        _parallel(6, 6, 10, 17, 0.7, None, [1.0, 0.05, 0.9, 0.999], 5, 9, 33),
    ],
}

# head sizes that the bfloat16 path takes to the tensor cores: chunk attention of 64 and 128 (prompt portions on the
# tensor-memory kernel, single tokens on the split kernel), matrix memories and recurrences of a few whole tiles
CONFIG_C = {
    "architecture": "Dedizen", "vocab": 160, "width": 64, "norm": {"eps": 3e-6},
    "layers": [
        _parallel(4, 2, 64, 21, 0.2, _rot(32, 10000.0, (8.0, 256, 16.0, 1.0)), [0.9, 0.98], 16, 32, 128),
        _mlstm(2, 32, 64, 15.0, 64),
        _rglru(128, 2, 4, 96),
        _parallel(2, 1, 128, 70, 0.12, _rot(128, 5000.0, (2.0, 512, 32.0, 1.0)), [0.6, 0.99, 0.999], 32, 16, None),
        _mlstm(3, 64, 80, 8.0, 32),
    ],
}

# one of everything that a model may happen to make equal or one
CONFIG_D = {
    "architecture": "Dedizen", "vocab": 64, "width": 40, "norm": {"eps": 2e-6},
    "layers": [
        _parallel(1, 1, 8, 1, 0.6, _rot(2, 30.0, (1.0, 32, 4.0, 2.0)), [0.8], 1, 1, 16),
        _mlstm(1, 1, 1, 1.0, 8),
        _rglru(8, 2, 2, 8),
        _parallel(2, 2, 18, 40, 0.3, _rot(6, 50.0), [0.97, 0.9], 8, 8, None),
    ],
}

# recurrences only: a model that keeps no paged cache at all, only states
CONFIG_E = {
    "architecture": "Dedizen", "vocab": 77, "width": 36, "norm": {"eps": 1e-5},
    "layers": [_rglru(40, 4, 4, 20), _mlstm(2, 12, 20, 12.0, None), _rglru(24, 2, 2, None)],
}

CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D, "E": CONFIG_E}


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """``name -> bfloat16 tensor`` for every tensor the configuration implies (names built here from the configuration
    alone, so the engine's own manifest is checked against an independent one)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def rnd(*shape, std=1.0):
        return torch.randn(*shape, generator=g) * std

    def lin(out, inn, gain=1.0):
        return rnd(out, inn, std=gain / math.sqrt(inn))

    def norm(n):
        return 1.0 + rnd(n, std=0.2)

    w: Dict[str, torch.Tensor] = {"embed": rnd(cfg["vocab"], W, std=0.6), "final.norm": norm(W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        w[p + "norm1"] = norm(W)
        if L["type"] == "mlstm":
            H, d, e = m["heads"], m["dim"], m["vdim"]
            w[q + "q"], w[q + "k"], w[q + "v"] = lin(H * d, W, 2.0), lin(H * d, W), lin(H * e, W)
            w[q + "g"], w[q + "o"], w[q + "norm"] = lin(H * e, W, 2.0), lin(W, H * e, 1.5), norm(H * e)
            w[q + "i"], w[q + "i.b"] = lin(H, W, 1.5), rnd(H, std=1.0)
            w[q + "f"], w[q + "f.b"] = lin(H, W, 1.5), 2.0 + rnd(H, std=1.0)
        elif L["type"] == "rglru":
            C, B = m["width"], m["blocks"]
            n = C // B
            w[q + "y"], w[q + "y.b"], w[q + "x"], w[q + "x.b"] = lin(C, W, 1.5), rnd(C, std=0.5), lin(C, W), rnd(C, std=0.5)
            w[q + "conv"], w[q + "conv.b"] = rnd(C, m["conv"], std=0.6), rnd(C, std=0.3)
            for r in ("ra", "ri"):
                w[q + r], w[q + r + ".b"] = rnd(B, n, n, std=1.5 / math.sqrt(n)), rnd(B, n, std=0.7)
            w[q + "lam"], w[q + "o"] = rnd(C, std=1.5) - 3.0, lin(W, C, 1.5)
        else:
            q, a = p + "mix.left.", m["left"]
            H, G, d = a["heads"], a["kv_heads"], a["dim"]
            w[q + "q"], w[q + "q.b"], w[q + "k"], w[q + "k.b"] = lin(H * d, W), rnd(H * d, std=0.5), lin(G * d, W), rnd(G * d, std=0.5)
            w[q + "sink"], w[q + "g"], w[q + "o"] = rnd(H, std=1.0), lin(H, W, 2.0), lin(W, H * d)
            w[q + "out"] = norm(W)
            q, r = p + "mix.right.", m["right"]
            H, d, e = r["heads"], r["dim"], r["vdim"]
            w[q + "q"], w[q + "k"], w[q + "v"] = lin(H * d, W, 1.5), lin(H * d, W, 1.5), lin(H * e, W, 1.5)
            w[q + "g"], w[q + "o"], w[q + "norm"] = lin(H * e, W, 2.0), lin(W, H * e), norm(H * e)
            w[q + "out"] = norm(W)
        if L.get("mlp") is not None:
            w[p + "norm2"] = norm(W)
            w[p + "mlp.up"], w[p + "mlp.down"] = lin(L["mlp"]["ff"], W, 1.2), lin(W, L["mlp"]["ff"])
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
