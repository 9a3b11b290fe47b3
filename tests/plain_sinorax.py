"""Sinorax, stated plainly: one slow function per mechanism, whole sequences, no cache, no batching.

Nothing here is shared with the package: the functions take the raw ``config.json`` dictionary and a dictionary of
checkpoint tensors by name, and work on one sequence ``[T, width]`` at a time in the dtype they are given (float64 for
an oracle that rounding does not touch). The attention builds its mask as a matrix and its weights one head at a time.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------------------------------------------------ small pieces
def dynamic_tanh(x, W: Dict[str, torch.Tensor], name: str):
    """tanh(alpha x) * w + b, element by element; alpha is one number per norm."""
    return torch.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def gelu_erf(z):
    """z times the normal distribution's share below z."""
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def cap_tanh(x, cap: Optional[float]):
    return x if not cap else cap * torch.tanh(x / cap)


# ------------------------------------------------------------------------------------------------------------ embedding
def bigram_row(previous: Optional[int], token: int, bigram: dict) -> int:
    """Row of the bigram table; a sequence's first token has the row behind the last bucket."""
    if previous is None:
        return int(bigram["buckets"])
    return (int(previous) * int(bigram["mul_prev"]) + int(token) * int(bigram["mul_cur"])) % int(bigram["buckets"])


def embed(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int]):
    x = W["embed"][torch.tensor(tokens)]
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram:
        rows = [bigram_row(tokens[i - 1] if i else None, t, bigram) for i, t in enumerate(tokens)]
        x = x + W["bigram"][torch.tensor(rows)]
    return x


# ------------------------------------------------------------------------------------------------------------ rotation
def turn_halves(x, angles):
    """x [T, heads, n], angles [T, n / 2]: the pair (m, m + n/2) turns by angle m."""
    half = x.shape[-1] // 2
    cos, sin = torch.cos(angles)[:, None, :], torch.sin(angles)[:, None, :]
    u, v = x[..., :half], x[..., half:]
    return torch.cat([u * cos - v * sin, v * cos + u * sin], dim=-1)


def angles_of(T: int, base: float, dims: int, factor: float, dtype):
    f = torch.tensor([base ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=torch.float64).to(dtype)
    return torch.arange(T).to(dtype)[:, None] * f[None, :]


def rotate_keys(x, rot: dict):
    """The first rot.dims entries of every head turn (slowed down by the scaling factor), the rest pass."""
    dims = int(rot["dims"])
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    a = angles_of(x.shape[0], float(rot["base"]), dims, factor, x.dtype)
    return torch.cat([turn_halves(x[..., :dims], a), x[..., dims:]], dim=-1)


def rotate_values(x, base: float, back: bool = False):
    """All entries turn with the token's position, at the plain frequencies; ``back``: the other way."""
    a = angles_of(x.shape[0], base, x.shape[-1], 1.0, x.dtype)
    return turn_halves(x, -a if back else a)


# ------------------------------------------------------------------------------------------------------------ attention
def projections(m: dict, W: Dict[str, torch.Tensor], p: str, h, bias: bool):
    T = h.shape[0]
    H, G, D, DV = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    out = []
    for name, heads, size in (("q", H, D), ("k", G, D), ("v", G, DV)):
        y = h @ W[f"{p}.{name}"].T
        if bias:
            y = y + W[f"{p}.{name}.b"]
        out.append(y.view(T, heads, size))
    return out


def rotated_attention(m: dict, W: Dict[str, torch.Tensor], p: str, h):
    """Causal softmax attention; queries and keys turn, values turn with their position and the result turns back."""
    T, H, G = h.shape[0], int(m["heads"]), int(m["kv_heads"])
    q, k, v = projections(m, W, p, h, bias=True)
    q, k = rotate_keys(q, m["rot"]), rotate_keys(k, m["rot"])
    base = float(m["rot"]["base"])
    v = rotate_values(v, base)
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    heads = []
    for n in range(H):
        g = n // (H // G)
        s = (q[:, n] @ k[:, g].T) * float(m["scale"])
        a = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1)
        heads.append(a @ v[:, g])
    o = rotate_values(torch.stack(heads, dim=1), base, back=True)
    return o.reshape(T, -1) @ W[p + ".o"].T + W[p + ".o.b"]


def sigmoid_attention(m: dict, W: Dict[str, torch.Tensor], p: str, h):
    """A sliding window whose keys are weighted by a sigmoid each, without a sum over keys; far keys score lower by the
    logarithm of their distance."""
    T, H, G = h.shape[0], int(m["heads"]), int(m["kv_heads"])
    q, k, v = projections(m, W, p, h, bias=False)
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = dist >= 0
    if m.get("mask"):
        seen = seen & (dist < int(m["mask"]["size"]))
    d = dist.clamp(min=0).to(h.dtype)
    heads = []
    for n in range(H):
        g = n // (H // G)
        s = (q[:, n] @ k[:, g].T) * float(m["scale"]) - W[p + ".r1"][n] * torch.log(1.0 + W[p + ".r2"][n] * d)
        a = torch.where(seen, torch.sigmoid(s + W[p + ".pb"][n]), torch.zeros_like(s))
        heads.append(a @ v[:, g])
    return torch.stack(heads, dim=1).reshape(T, -1) @ W[p + ".o"].T


MIXERS = {"attention": rotated_attention, "attention_2": sigmoid_attention}


# ------------------------------------------------------------------------------------------------------------ the model
def feed_forward(W: Dict[str, torch.Tensor], p: str, h):
    return gelu_erf(h @ W[p + ".up"].T) @ W[p + ".down"].T


def layer(cfg: dict, W: Dict[str, torch.Tensor], i: int, x):
    lc, p = cfg["layers"][i], f"l{i}"
    x = x + dynamic_tanh(MIXERS[lc["type"]](lc["mixer"], W, f"{p}.mix", dynamic_tanh(x, W, f"{p}.norm1")), W, f"{p}.norm1b")
    if lc.get("mlp"):
        x = x + dynamic_tanh(feed_forward(W, f"{p}.mlp", dynamic_tanh(x, W, f"{p}.norm2")), W, f"{p}.norm2b")
    return x


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64, streams: Optional[list] = None):
    """Logits [T, vocab]; ``streams`` collects the residual after every layer."""
    W = {k: v.to(dtype) for k, v in tensors.items()}
    x = embed(cfg, W, list(tokens))
    for i in range(len(cfg["layers"])):
        x = layer(cfg, W, i, x)
        if streams is not None:
            streams.append(x.clone())
    logits = dynamic_tanh(x, W, "final.norm") @ W["head"].T * float(cfg.get("logit_scale", 1.0))
    return cap_tanh(logits, cfg.get("logit_softcap"))
