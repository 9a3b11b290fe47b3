"""Sinorax: a decoder whose layers are listed one by one in config.json.

A Dynamic Tanh (``tanh(alpha x) w + b``, no mean, no variance) stands before every sublayer and another on its result:
``x += norm1b(mixer(norm1(x)))``, then ``x += norm2b(ff(norm2(x)))`` where the layer has a feed-forward (dense, exact GELU). The mixer
is one of

* ``attention``: grouped causal softmax attention with biases; queries and keys turn in pairs half the rotated entries apart, at
  frequencies that a factor slows down; values turn too, over all their entries at the plain frequencies, are cached so, and each
  head's result turns back by its own position;
* ``attention_2``: a sliding window without rotation; a penalty ``r1 ln(1 + r2 distance)`` per head, and sigmoid weights that are
  not normalised over the keys.

To a token's embedding a row of a bigram table is added, chosen by the token and the one before it (a request's last token is
part of its state). The logits have a head of their own, a factor and a soft cap.
Tensor names: ``embed``, ``bigram``, ``l<i>.norm1/norm1b/norm2/norm2b`` (each with ``.b`` and ``.alpha``), ``l<i>.mix.q/k/v/o`` (``.b``),
``l<i>.mix.r1/r2/pb``, ``l<i>.mlp.up/down``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.model_config import SinoraxConfig
from ..parts import OutputHead, TokenEmbedding
from ..parts.attention_masked import MaskedAttention
from ..parts.block import SandwichBlock
from ..parts.embedding import BigramEmbedding
from ..parts.mlp import DenseMLP
from ..parts.norm import DynamicTanh
from ..parts.rotary import LinearRotary
from .registry import register_architecture
from .spec import ModelSpec, sequential


def build_sinorax(cfg: SinoraxConfig) -> ModelSpec:
    W = cfg.width
    layers = []
    for i, lc in enumerate(cfg.layers):
        p, m = f"l{i}", lc.mixer
        if lc.kind == "attention":
            r = m.rot
            mixer = MaskedAttention(W, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, f"{p}.mix", position=LinearRotary(r.dims, r.base, r.factor),
                                    bias=True, value_position=LinearRotary(m.vdim, r.base))
        else:
            mixer = MaskedAttention(W, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, f"{p}.mix", window=m.window, log_distance=True,
                                    scoring="sigmoid")
        ff = DenseMLP(W, lc.ff, f"{p}.mlp.up", f"{p}.mlp.down", "gelu_erf") if lc.ff else None
        layers.append(SandwichBlock(DynamicTanh(W, f"{p}.norm1"), mixer, DynamicTanh(W, f"{p}.norm1b"),
                                    DynamicTanh(W, f"{p}.norm2") if ff else None, ff, DynamicTanh(W, f"{p}.norm2b") if ff else None))
    b = cfg.bigram
    embedding = BigramEmbedding(cfg.vocab, W, "embed", "bigram", b.buckets, b.mul_prev, b.mul_cur) if b else TokenEmbedding(cfg.vocab, W, "embed")
    return ModelSpec(
        config=cfg,
        embedding=embedding,
        layers=layers,
        schedule=sequential(len(layers)),
        final_norm=DynamicTanh(W, "final.norm"),
        head=OutputHead(cfg.vocab, W, "head", softcap=cfg.logit_softcap, scale=cfg.logit_scale),
    )


register_architecture("Sinorax", SinoraxConfig, build_sinorax)
