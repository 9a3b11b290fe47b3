"""Putelix: a decoder whose layers are listed one by one in config.json.

The sublayers read the residual stream itself and their results are normed before they are added: ``x += norm1(mixer(x))``, then
``x += norm2(ff(x))`` where the layer has a feed-forward (RMS norms with plain weights). The mixer is ``parallel``, half the sum of
two results that are normed over the model width each:

* left: grouped causal attention within chunks of positions; queries and keys are normed as whole projections, the values are the
  keys before that norm, scores are soft-capped and then biased by bucketed distance, every head has an output gate;
* right: linear attention with a fixed decay per head (a recurrent state of fixed size), its heads normed together and gated.

The feed-forward is a dense unit with squared relu, or routed experts (the largest logits, weighted by the softmax over them alone)
with a shared expert behind a gate per token, or absent. A learned vector per position is added to a token's embedding; the output
head is the embedding table itself.
Tensor names: ``embed``, ``pos``, ``l<i>.norm1/norm2``, ``l<i>.mix.left.*``, ``l<i>.mix.right.*``, ``l<i>.mlp.*``, ``final.norm``.
"""
from __future__ import annotations

from ..config.model_config import PutelixConfig, TopSoftmaxExpertsConfig
from ..parts import OutputHead
from ..parts.attention_masked import MaskedAttention
from ..parts.block import PostNormBlock
from ..parts.embedding import PositionedEmbedding
from ..parts.mlp import DenseMLP, GatedUnit, RoutedExperts
from ..parts.norm import RMSNorm
from ..parts.recurrent import DecayedLinearAttention, ParallelMixer
from .registry import register_architecture
from .spec import ModelSpec, sequential


def build_putelix(cfg: PutelixConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.eps

    def feed_forward(mlp, p: str):
        if mlp is None:
            return None
        if isinstance(mlp, TopSoftmaxExpertsConfig):
            shared = GatedUnit(W, mlp.shared_ff, f"{p}.shared.gate", f"{p}.shared.up", f"{p}.shared.down", "silu") if mlp.shared_ff else None
            return RoutedExperts(W, mlp.ff, mlp.experts, 0, mlp.top, p, shared, scoring="top_softmax", correction=False, router_bias=True,
                                 shared_gate=f"{p}.shared.sg" if shared else None)
        return DenseMLP(W, int(mlp), f"{p}.up", f"{p}.down", "relu2")

    layers = []
    for i, lc in enumerate(cfg.layers):
        p, a, r = f"l{i}", lc.mixer.left, lc.mixer.right
        left = MaskedAttention(W, a.heads, a.kv_heads, a.dim, a.dim, a.scale, f"{p}.mix.left", chunk=a.chunk, softcap=a.softcap, qk_norm="rows",
                               eps=eps, values_are_keys=True, bias=True, head_gate=True, bias_far=a.bias_max)
        right = DecayedLinearAttention(W, r.heads, r.dim, r.vdim, r.decay, eps, f"{p}.mix.right")
        mixer = ParallelMixer(W, left, right, eps, f"{p}.mix.left.out", f"{p}.mix.right.out")
        ff = feed_forward(lc.mlp, f"{p}.mlp")
        layers.append(PostNormBlock(mixer, RMSNorm(W, eps, f"{p}.norm1"), ff, RMSNorm(W, eps, f"{p}.norm2") if ff else None))
    embedding = PositionedEmbedding(cfg.vocab, W, "embed", "pos", cfg.max_positions)
    return ModelSpec(
        config=cfg,
        embedding=embedding,
        layers=layers,
        schedule=sequential(len(layers)),
        final_norm=RMSNorm(W, eps, "final.norm"),
        head=OutputHead(cfg.vocab, W, "head", tied_to=embedding),
    )


register_architecture("Putelix", PutelixConfig, build_putelix)
