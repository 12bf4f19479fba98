"""A plain, slow Dedizen: one function per mechanism, float64 on the CPU, written from the design's equations and
sharing no code with the engine.

``forward(config, weights, tokens)`` runs one whole sequence and returns the logits ``[T, V]`` (with ``layers_out``, a
list, the residual stream after every layer is appended to it).  ``weights`` maps checkpoint names to tensors.  With
``rnd`` (a function that rounds a tensor, ``as_bfloat16``) the places where the engine's bfloat16 path stores 16 bits
are rounded too, so that a tiny model's own sensitivity to rounding does not drown a comparison.
"""

from __future__ import annotations

import math
from typing import Callable, Dict, Optional

import torch

F64 = torch.float64


def as_bfloat16(x: torch.Tensor) -> torch.Tensor:
    return x.to(torch.bfloat16).to(x.dtype)


def same(x: torch.Tensor) -> torch.Tensor:
    return x


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.where(x > 30.0, x, torch.log1p(torch.exp(torch.clamp(x, max=30.0))))


def log_sigmoid(x):
    return -softplus(-x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """The last dimension divided by its root mean square."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def causal_conv(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """``y_t = b + sum_j w[:, j] x_(t - taps + 1 + j)`` per channel, zeros before the sequence."""
    T, C = x.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x], dim=0)
    y = torch.zeros_like(x) + b
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


# --------------------------------------------------------------------------- #
# matrix memory with exponential gates
# --------------------------------------------------------------------------- #

def matrix_memory(q, k, v, i, f):
    """``q, k [T, H, d]``, ``v [T, H, e]``, log gates ``i, f [T, H]`` -> ``[T, H, e]``.  The memory and the sum of its
    keys are kept divided by ``exp(m)``, ``m`` a running maximum that starts at 0."""
    T, H, d = k.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=v.dtype)
    n = torch.zeros(H, d, dtype=v.dtype)
    m = torch.zeros(H, dtype=v.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=v.dtype)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        m = m_new
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        denom = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hkv,hk->hv", S, q[t]) / denom[:, None]
    return out


def mlstm_mixer(h, W, p, m, eps, rnd):
    T = h.shape[0]
    H, d, e, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = rnd(h @ W[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = rnd(h @ W[p + "k"].T).reshape(T, H, d)
    v = rnd(h @ W[p + "v"].T).reshape(T, H, e)
    i = cap * torch.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap))
    o = unit_rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * e) * W[p + "norm"]
    return rnd(o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# --------------------------------------------------------------------------- #
# gated linear recurrence per channel
# --------------------------------------------------------------------------- #

def block_product(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """``u [T, blocks * n]``, ``w [blocks, n, n]`` (``[out, in]``), ``b [blocks, n]``: every part with its own matrix."""
    blocks, n = w.shape[0], w.shape[1]
    parts = u.reshape(u.shape[0], blocks, n)
    return (torch.einsum("tbi,boi->tbo", parts, w) + b).reshape(u.shape[0], blocks * n)


def real_gated_lru(u, r, i, lam):
    """``u, r, i [T, C]``, ``lam [C]``: ``a = exp(-8 r softplus(lam))``, ``S <- a S + sqrt(1 - a^2) i u``."""
    log_a = -8.0 * r * softplus(lam)
    a, drive = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    S = torch.zeros(u.shape[1], dtype=u.dtype)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + drive[t]
        out[t] = S
    return out


def rglru_mixer(h, W, p, m, eps, rnd):
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = causal_conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    r = sigmoid(block_product(u, W[p + "ra"], W[p + "ra.b"]))
    i = sigmoid(block_product(u, W[p + "ri"], W[p + "ri.b"]))
    return rnd(real_gated_lru(u, r, i, W[p + "lam"]) * y) @ W[p + "o"].T


# --------------------------------------------------------------------------- #
# attention inside chunks, beside linear attention with fixed decays
# --------------------------------------------------------------------------- #

def yarn(dims: int, rot: dict):
    """Frequencies per pair and the factor on cosines and sines."""
    base = rot["base"]
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if s is None:
        return freq, 1.0

    def dim(t):
        return dims * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim(s["fast"])), 0), min(math.ceil(dim(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """``x [T, heads, d]``: of the first ``dims`` dimensions ``2i`` turns with ``2i + 1``."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    freq, mag = yarn(dims, rot)
    ang = positions.to(x.dtype)[:, None] * torch.tensor(freq, dtype=x.dtype)[None, :]
    c, s = mag * torch.cos(ang)[:, None, :], mag * torch.sin(ang)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


def sink_softmax(score: torch.Tensor, visible: torch.Tensor, sink) -> torch.Tensor:
    """Rows of ``score`` over the visible keys; the denominator holds ``exp(sink)`` as well."""
    score = torch.where(visible, score, torch.full_like(score, -math.inf))
    top = torch.maximum(score.max(dim=-1, keepdim=True).values, sink)
    e = torch.exp(score - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def chunk_attention(h, W, p, m, eps, rnd):
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).reshape(T, H, d)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).reshape(T, G, d)
    v = rnd(k)
    pos = torch.arange(T)
    q = rnd(unit_rms(rotate_neighbours(q, pos, m.get("rot")), eps))
    k = rnd(unit_rms(rotate_neighbours(k, pos, m.get("rot")), eps))
    i, j = pos[:, None], pos[None, :]
    size = m["mask"]["size"]
    visible = (j <= i) & (i // size == j // size)
    out = torch.zeros(T, H, d, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = rnd(sink_softmax((q[:, hd] @ k[:, g].T) * m["scale"], visible, W[p + "sink"][hd])) @ v[:, g]
    gate = sigmoid(h @ W[p + "g"].T)
    return rnd(out * gate[:, :, None]).reshape(T, H * d) @ W[p + "o"].T


def fixed_decay_memory(q, k, v, decay):
    """``S <- decay_h S + k v^T``, ``o = S^T q`` per head."""
    T, H, d = k.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=v.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=v.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out


def lightning_attention(h, W, p, m, eps, rnd):
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q, k = rnd(silu(h @ W[p + "q"].T)).reshape(T, H, d), rnd(silu(h @ W[p + "k"].T)).reshape(T, H, d)
    v = rnd(silu(h @ W[p + "v"].T)).reshape(T, H, e)
    o = fixed_decay_memory(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)).reshape(T, H * e)
    return rnd(unit_rms(o, eps) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel_mixer(h, W, p, m, eps, rnd):
    left = chunk_attention(h, W, p + "left.", m["left"], eps, rnd)
    right = lightning_attention(h, W, p + "right.", m["right"], eps, rnd)
    return 0.5 * (unit_rms(left, eps) * W[p + "left.out"] + unit_rms(right, eps) * W[p + "right.out"])


MIXERS = {"mlstm": mlstm_mixer, "rglru": rglru_mixer, "parallel": parallel_mixer}


def feed_forward(h, W, p, rnd):
    return rnd(torch.relu(rnd(h @ W[p + "up"].T)) ** 2) @ W[p + "down"].T


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens, rnd: Optional[Callable] = None,
            layers_out: Optional[list] = None, dtype: torch.dtype = F64) -> torch.Tensor:
    """``dtype`` float32 runs the same plain arithmetic in 32 bits: how far it lies from the float64 run says how much
    rounding alone moves a position of THIS model."""
    rnd = rnd or same
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](rnd(unit_rms(x, eps) * W[p + "norm1"]), W, p + "mix.", layer["mixer"], eps, rnd)
        if layer.get("mlp") is not None:
            x = x + feed_forward(rnd(unit_rms(x, eps) * W[p + "norm2"]), W, p + "mlp.", rnd)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rnd(unit_rms(x, eps) * W["final.norm"]) @ W["embed"].T


def greedy(config: dict, weights: Dict[str, torch.Tensor], prompt, n: int):
    ids, out = list(prompt), []
    for _ in range(n):
        tok = int(torch.argmax(forward(config, weights, ids)[-1]))
        ids.append(tok)
        out.append(tok)
    return out
