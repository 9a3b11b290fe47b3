"""Putelix, stated plainly: one slow function per mechanism, whole sequences, no cache, no batching.

Nothing here is shared with the package: the functions take the raw ``config.json`` dictionary and a dictionary of
checkpoint tensors by name, and work on one sequence ``[T, width]`` at a time in the dtype they are given (float64 for
an oracle that rounding does not touch). The attention builds mask and bias as matrices, one head at a time; the
recurrence is a loop over the tokens; every expert runs by itself.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------------------------------------------------ small pieces
def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def cap_tanh(x, cap: Optional[float]):
    return x if not cap else cap * torch.tanh(x / cap)


# ------------------------------------------------------------------------------------------------------------ embedding
def embed(W: Dict[str, torch.Tensor], tokens: List[int]):
    """A token's row plus the row of its position, neither of them scaled."""
    return W["embed"][torch.tensor(tokens)] + W["pos"][: len(tokens)]


# ------------------------------------------------------------------------------------------------------------ attention
def bucket(n: int, rows: int, far: float) -> int:
    """Row of the distance table: one per distance for the first half, then logarithmically wider up to ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def distance_bias(rel, T: int, far: float):
    """[heads, T, T]: entry (h, i, j) is the bias of query i for key j <= i (zero elsewhere)."""
    rows = torch.tensor([[bucket(max(i - j, 0), rel.shape[0], far) for j in range(T)] for i in range(T)])
    return rel[rows].permute(2, 0, 1)


def chunk_mask(T: int, size: Optional[int]):
    """True where query i sees key j: not later, and in the same run of ``size`` positions."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if not size else seen & (i // size == j // size)


def chunked_attention(m: dict, W: Dict[str, torch.Tensor], p: str, h, eps: float):
    """Queries and keys normed as whole projections; the values are the keys before that norm; scores scaled, capped, then
    biased by distance; a gate per head."""
    T, H, G, D = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = h @ W[f"{p}.q"].T + W[f"{p}.q.b"]
    k = h @ W[f"{p}.k"].T + W[f"{p}.k.b"]
    v = k.view(T, G, D)
    q = rms_norm(q, W[f"{p}.q.norm"], eps).view(T, H, D)
    k = rms_norm(k, W[f"{p}.k.norm"], eps).view(T, G, D)
    gate = torch.sigmoid(h @ W[f"{p}.g"].T)
    bias = distance_bias(W[f"{p}.rel"], T, float(m["bias_max"]))
    seen = chunk_mask(T, (m.get("mask") or {}).get("size"))
    heads = []
    for n in range(H):
        g = n // (H // G)
        s = cap_tanh((q[:, n] @ k[:, g].T) * float(m["scale"]), m.get("softcap")) + bias[n]
        a = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1)
        heads.append((a @ v[:, g]) * gate[:, n:n + 1])
    return torch.cat(heads, dim=1) @ W[f"{p}.o"].T + W[f"{p}.o.b"]


# ------------------------------------------------------------------------------------------------------------ linear attention
def lightning_attention(m: dict, W: Dict[str, torch.Tensor], p: str, h, eps: float):
    """Per head S <- decay S + k v^T, o = S^T q; the heads normed together, gated, projected."""
    T, H, D, DV = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(h @ W[f"{p}.q"].T).view(T, H, D)
    k = silu(h @ W[f"{p}.k"].T).view(T, H, D)
    v = silu(h @ W[f"{p}.v"].T).view(T, H, DV)
    out = h.new_zeros(T, H, DV)
    for n in range(H):
        S = h.new_zeros(D, DV)
        for t in range(T):
            S = float(m["decay"][n]) * S + torch.outer(k[t, n], v[t, n])
            out[t, n] = S.T @ q[t, n]
    y = rms_norm(out.reshape(T, H * DV), W[f"{p}.norm"], eps) * torch.sigmoid(h @ W[f"{p}.g"].T)
    return y @ W[f"{p}.o"].T


def parallel_mixer(m: dict, W: Dict[str, torch.Tensor], p: str, h, eps: float):
    left = chunked_attention(m["left"], W, f"{p}.left", h, eps)
    right = lightning_attention(m["right"], W, f"{p}.right", h, eps)
    return 0.5 * (rms_norm(left, W[f"{p}.left.out"], eps) + rms_norm(right, W[f"{p}.right.out"], eps))


# ------------------------------------------------------------------------------------------------------------ feed-forward
def dense_unit(W: Dict[str, torch.Tensor], p: str, h):
    """down(relu(up x)^2)"""
    return torch.clamp(h @ W[f"{p}.up"].T, min=0) ** 2 @ W[f"{p}.down"].T


def gated_unit(W: Dict[str, torch.Tensor], p: str, h):
    return (silu(h @ W[f"{p}.gate"].T) * (h @ W[f"{p}.up"].T)) @ W[f"{p}.down"].T


def route(logits, top: int):
    """The ``top`` largest logits; their weights are the softmax over the chosen ones alone."""
    values, ids = torch.topk(logits, top, dim=-1)
    return ids, torch.softmax(values, dim=-1)


def routed_experts(mlp: dict, W: Dict[str, torch.Tensor], p: str, h, forced=None, regret_out: Optional[list] = None):
    """``forced [T, top]``: these experts are taken instead of the router's own choice (their weights are still the softmax over the
    router's logits for them); ``regret_out`` then collects, per token, how far the smallest logit taken lies below the smallest of the
    router's own choice."""
    logits = h @ W[f"{p}.router"].T + W[f"{p}.router.b"]
    ids, weights = route(logits, int(mlp["router"]["top"]))
    if forced is not None:
        taken = logits.gather(1, forced)
        if regret_out is not None:
            regret_out.append(logits.gather(1, ids).min(-1).values - taken.min(-1).values)
        ids, weights = forced, torch.softmax(taken, dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(ids[t].tolist(), weights[t]):
            out[t] += w * gated_unit(W, f"{p}.e{e}", h[t:t + 1])[0]
    if mlp.get("shared"):
        out = out + gated_unit(W, f"{p}.shared", h) * torch.sigmoid(h @ W[f"{p}.shared.sg"].T)
    return out


# ------------------------------------------------------------------------------------------------------------ the model
def layer(cfg: dict, W: Dict[str, torch.Tensor], i: int, x, forced: Optional[list] = None, regret_out: Optional[list] = None):
    lc, p, eps = cfg["layers"][i], f"l{i}", float(cfg["norm"]["eps"])
    x = x + rms_norm(parallel_mixer(lc["mixer"], W, f"{p}.mix", x, eps), W[f"{p}.norm1"], eps)
    mlp = lc.get("mlp")
    if mlp:
        y = routed_experts(mlp, W, f"{p}.mlp", x, forced.pop(0) if forced else None, regret_out) if mlp["kind"] == "moe" else dense_unit(W, f"{p}.mlp", x)
        x = x + rms_norm(y, W[f"{p}.norm2"], eps)
    return x


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64, streams: Optional[list] = None,
            forced: Optional[list] = None, regret_out: Optional[list] = None):
    """Logits [T, vocab]; ``streams`` collects the residual after every layer. ``forced`` (a list over the layers with experts of ``[T, top]``):
    the experts to take instead of the routers' own choice, what another implementation chose, so that the two can be compared where
    a choice hung on rounding."""
    W = {k: v.to(dtype) for k, v in tensors.items()}
    x = embed(W, list(tokens))
    forced = list(forced) if forced else None
    for i in range(len(cfg["layers"])):
        x = layer(cfg, W, i, x, forced, regret_out)
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, W["final.norm"], float(cfg["norm"]["eps"])) @ W["embed"].T
