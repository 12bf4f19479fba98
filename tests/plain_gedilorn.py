"""A plain, slow Gedilorn in PyTorch on the CPU: one function per mechanism, whole sequences at once, no
cache and no state carried between calls.  It shares no code with the engine and is what the engine's kernels,
parts and step function are compared with.  ``dtype`` float64 gives an oracle whose own rounding is far below
the float32 engine's.

Notation: ``T`` tokens, ``W`` width, ``S`` residual streams, ``H`` heads, ``d`` / ``r`` plain and rotated
query/key sizes of a head, ``e`` value size, ``c`` latent size.  Weights are a dict ``name -> tensor`` with the
checkpoint's names; a configuration is the dictionary of ``config.json``.
"""

from __future__ import annotations

import math
from typing import Callable, Dict, List, Optional

import torch


def same(t):
    return t


def as_bfloat16(t):
    """Round to bfloat16 and back: handed to ``forward`` as ``rnd`` it rounds where the engine's bfloat16
    path stores 16 bits (the inputs of its matrix products and the cache)."""
    return t.to(torch.bfloat16).to(t.dtype)


# --------------------------------------------------------------------------- #
# norm
# --------------------------------------------------------------------------- #

def rms_norm(x, w, eps: float):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps) * w


# --------------------------------------------------------------------------- #
# embedding
# --------------------------------------------------------------------------- #

def bigram_rows(tokens: List[int], bigram: dict) -> List[int]:
    """The table row of every place: a hash of the token before it and the token itself; the table's last row
    at a sequence's start."""
    n, a, b = int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"])
    return [n if i == 0 else (tokens[i - 1] * a + t * b) % n for i, t in enumerate(tokens)]


def embedding_output(config: dict, w: Dict[str, torch.Tensor], tokens: List[int]):
    emb = config["embedding"]
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * float(emb["scale"])
    x = x + w["bigram"][torch.tensor(bigram_rows(tokens, emb["bigram"]), dtype=torch.long)]
    return rms_norm(x, w["embed.norm"], float(config["norm"]["eps"]))


# --------------------------------------------------------------------------- #
# rotation
# --------------------------------------------------------------------------- #

def yarn_frequencies(dims: int, base: float, scaling: Optional[dict]):
    """``(frequency of every pair (list of dims / 2), factor on cos and sin)``."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def dim_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(dim_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_neighbours(x, freqs: List[float], magnitude: float):
    """``x [T, heads, r]``: coordinate ``2i`` is paired with ``2i + 1``; the pair turns by ``position *
    freqs[i]`` and is stretched by ``magnitude``."""
    T, n = x.shape[0], len(freqs)
    a = torch.arange(T, dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)[None, :]
    cos, sin = (torch.cos(a) * magnitude).to(x.dtype)[:, None, :], (torch.sin(a) * magnitude).to(x.dtype)[:, None, :]
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out = x.clone()
    out[..., 0:2 * n:2] = u * cos - v * sin
    out[..., 1:2 * n:2] = v * cos + u * sin
    return out


# --------------------------------------------------------------------------- #
# attention through a latent
# --------------------------------------------------------------------------- #

def causal_softmax_attention(q, k, v, scale: float):
    """``q, k [T, H, *]``, ``v [T, H, e]`` -> ``[T, H, e]``; a query sees itself and everything before it."""
    T, H, _ = q.shape
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    out = []
    for h in range(H):
        s = ((q[:, h, :] @ k[:, h, :].T) * scale).masked_fill(~mask, float("-inf"))
        out.append(torch.softmax(s, dim=-1) @ v[:, h, :])
    return torch.stack(out, dim=1)


def latent_attention_mixer(h, w, p: str, m: dict, eps: float, gated: bool, rnd: Callable = same):
    """Every head's keys and values are formed from the latents; nothing is folded into the queries."""
    T = h.shape[0]
    H, d, r, e, c = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    freqs, magnitude = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    dkv = h @ w[p + "dkv"].T
    latent = rnd(rms_norm(dkv[:, :c], w[p + "dkv.norm"], eps))
    k_rot = rnd(rotate_neighbours(dkv[:, c:].reshape(T, 1, r), freqs, magnitude))
    k_plain = (latent @ w[p + "uk"].T).view(T, H, d)
    v = (latent @ w[p + "uv"].T).view(T, H, e)
    qq = torch.cat([rnd(q[..., :d]), rnd(rotate_neighbours(q[..., d:], freqs, magnitude))], dim=-1)
    kk = torch.cat([k_plain, k_rot.expand(T, H, r)], dim=-1)
    a = causal_softmax_attention(qq, kk, v, float(m["scale"])).reshape(T, H * e)
    if gated:
        a = a * torch.sigmoid(h @ w[p + "g"].T)
    return rnd(a) @ w[p + "o"].T


# --------------------------------------------------------------------------- #
# feed-forward
# --------------------------------------------------------------------------- #

def relu_glu_ff(h, w, p: str, rnd: Callable = same):
    return rnd(torch.relu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# --------------------------------------------------------------------------- #
# hyper-connections
# --------------------------------------------------------------------------- #

def streams_read(xs, w_in):
    """``xs [T, S, W]`` -> ``[T, W]``: what a sublayer reads."""
    return torch.einsum("s,tsw->tw", w_in, xs)


def streams_update(xs, mix, w_out, y):
    """``mix[from, to]``: all streams at once from the old ones, plus every stream's share of ``y``."""
    return torch.einsum("sr,tsw->trw", mix, xs) + w_out[None, :, None] * y[:, None, :]


# --------------------------------------------------------------------------- #
# the model
# --------------------------------------------------------------------------- #

def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            rnd: Callable = same, layers_out: Optional[list] = None):
    """Logits ``[T, vocab]`` of a whole sequence.  ``layers_out`` receives the sum of the streams after every
    run of a layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = embedding_output(config, w, tokens)
    xs = x[:, None, :].repeat(1, int(config["streams"]), 1)
    for i, layer in enumerate(config["layers"]):
        own = i
        while config["layers"][own].get("weights_of") is not None:
            own = config["layers"][own]["weights_of"]
        p = f"l{own}."
        h = rnd(rms_norm(streams_read(xs, w[p + "hc1.in"]), w[p + "norm1"], eps))
        y = latent_attention_mixer(h, w, p + "mix.", layer["mixer"], eps, layer["type"] == "latent_attention_2", rnd)
        xs = streams_update(xs, w[p + "hc1.mix"], w[p + "hc1.out"], y)
        if layer.get("mlp") is not None:
            h = rnd(rms_norm(streams_read(xs, w[p + "hc2.in"]), w[p + "norm2"], eps))
            xs = streams_update(xs, w[p + "hc2.mix"], w[p + "hc2.out"], relu_glu_ff(h, w, p + "mlp.", rnd))
        if layers_out is not None:
            layers_out.append(xs.sum(dim=1))
    x = rnd(rms_norm(xs.sum(dim=1), w["final.norm"], eps))
    return x @ w["head"].T * float(config["logit_scale"])


def greedy(config: dict, weights, prompt: List[int], n: int, dtype=torch.float64) -> List[int]:
    """``n`` tokens, each the arg-max of the logits at the last position of all tokens so far."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(torch.argmax(forward(config, weights, toks, dtype)[-1])))
    return toks[len(prompt):]
