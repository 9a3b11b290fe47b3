"""Token embedding and output head."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..cache.spec import FixedStateSpec
from .base import ANY, MATRIX, ParamSpec, Part, Source


class TokenEmbedding(Part):
    """``x = table[token] * scale`` (the reference has no scaling, src/miniserve/model.py:229), widened into the 32-bit
    residual stream; the product is taken in 32-bit."""

    graph_safe = True

    def __init__(self, vocab: int, hidden: int, name: str, scale: float = 1.0):
        self.vocab, self.hidden, self.name, self.scale = vocab, hidden, name, float(scale)
        self.table: Optional[torch.Tensor] = None

    def params(self) -> Dict[str, ParamSpec]:
        return {"table": ParamSpec((Source(self.name, (self.vocab, self.hidden)),), MATRIX)}

    def cache_spec(self):
        """What the embedding keeps per request (as a mixer's ``cache_spec``); nothing here."""
        return None

    def position_limit(self) -> Optional[int]:
        """The most positions a request may have, or None where the embedding sets no limit."""
        return None

    def forward(self, ctx, cache=None) -> torch.Tensor:
        if self.scale == 1.0:
            return ctx.K.embed(ctx.token_ids, self.table)
        return ctx.K.embed(ctx.token_ids, self.table, self.scale)

    def add_into(self, ctx, residual: torch.Tensor) -> None:
        """``residual += table[token] * scale``: the step's embedding once more, for a model that feeds it in again on the way."""
        ctx.K.embed_add(ctx.token_ids, self.table, residual, self.scale)


class PositionedEmbedding(TokenEmbedding):
    """``x = table[token] * scale + positions[p]`` for the token at position p of its request, the sum in 32-bit. ``max_positions`` rows
    (None: the checkpoint's tensor decides): no request can become longer than that."""

    def __init__(self, vocab: int, hidden: int, name: str, position_name: str, max_positions: Optional[int] = None, scale: float = 1.0,
                 random_positions: int = 256):
        super().__init__(vocab, hidden, name, scale)
        self.position_name, self.max_positions, self.random_positions = position_name, max_positions, int(random_positions)
        self.position_table: Optional[torch.Tensor] = None

    def params(self) -> Dict[str, ParamSpec]:
        rows = self.max_positions if self.max_positions else ANY
        return {**super().params(), "position_table": ParamSpec((Source(self.position_name, (rows, self.hidden), free=self.random_positions),), MATRIX)}

    def position_limit(self) -> Optional[int]:
        return self.max_positions if self.position_table is None else self.position_table.shape[0]

    def forward(self, ctx, cache=None) -> torch.Tensor:
        return ctx.K.embed_positions(ctx.token_ids, self.table, ctx.positions, self.position_table, self.scale)

    def add_into(self, ctx, residual: torch.Tensor) -> None:
        raise ValueError("an embedding with positions is not fed in again on the way")


class BigramEmbedding(TokenEmbedding):
    """``x = table[token] * scale + bigram[(previous * mul_prev + token * mul_cur) mod buckets]``; a request's first token, which has no
    previous one, takes the bigram table's last row, number ``buckets``. A request's last token is its state: a portion may
    start anywhere, and a decoded token may be known to the device alone."""

    def __init__(self, vocab: int, hidden: int, name: str, bigram_name: str, buckets: int, mul_prev: int, mul_cur: int, scale: float = 1.0):
        super().__init__(vocab, hidden, name, scale)
        if buckets < 1:
            raise ValueError(f"a bigram table needs at least one bucket, got {buckets}")
        self.bigram_name, self.buckets, self.mul_prev, self.mul_cur = bigram_name, int(buckets), int(mul_prev), int(mul_cur)
        self.bigram: Optional[torch.Tensor] = None

    def params(self) -> Dict[str, ParamSpec]:
        return {**super().params(), "bigram": ParamSpec((Source(self.bigram_name, (self.buckets + 1, self.hidden)),), MATRIX)}

    def cache_spec(self):
        return FixedStateSpec((1,), zeroed=False)

    def forward(self, ctx, cache=None) -> torch.Tensor:
        return ctx.K.embed_bigram(ctx.token_ids, self.table, self.bigram, self.buckets, self.mul_prev, self.mul_cur, ctx.positions, ctx.token_seq,
                                  ctx.seq_starts_dev, ctx.num_seqs, cache.state.view(torch.int32), self.scale)

    def add_into(self, ctx, residual: torch.Tensor) -> None:
        raise ValueError("a bigram embedding is not fed in again on the way")


class OutputHead(Part):
    """``logits = h W^T`` without bias, in 32-bit. ``tied_to`` makes ``W`` the embedding's own table
    (src/miniserve/model.py:204-206); a tensor of the head's name in the checkpoint is then not needed. The logits are multiplied by
    ``scale``; ``softcap`` then bounds them: ``softcap * tanh(logits / softcap)``."""

    graph_safe = True

    def __init__(self, vocab: int, hidden: int, name: str, tied_to: Optional[TokenEmbedding] = None, softcap: Optional[float] = None,
                 scale: float = 1.0):
        self.vocab, self.hidden, self.name, self.tied_to = vocab, hidden, name, tied_to
        self.softcap = float(softcap) if softcap else None
        self.scale = float(scale)
        self.weight: Optional[torch.Tensor] = None

    def params(self) -> Dict[str, ParamSpec]:
        if self.tied_to is not None:
            return {}
        return {"weight": ParamSpec((Source(self.name, (self.vocab, self.hidden)),), MATRIX)}

    def ignored_names(self):
        """Checkpoint names that may be present without being read."""
        return (self.name,) if self.tied_to is not None else ()

    def aliases(self) -> Dict[str, str]:
        """Ignored checkpoint name -> the tensor that stands in for it; the loader warns when the two differ."""
        return {self.name: self.tied_to.name} if self.tied_to is not None else {}

    def matrix(self) -> torch.Tensor:
        return self.tied_to.table if self.tied_to is not None else self.weight

    def forward(self, ctx, h: torch.Tensor) -> torch.Tensor:
        logits = ctx.K.linear(h, self.matrix(), out_dtype=torch.float32)
        if self.scale != 1.0:
            return ctx.K.softcap(logits, self.softcap, self.scale)
        return ctx.K.softcap(logits, self.softcap) if self.softcap else logits
