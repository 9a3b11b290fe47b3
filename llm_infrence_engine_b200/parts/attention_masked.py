"""Grouped-query attention with partly rotated heads and a mask that is more than causal."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..cache.spec import FixedStateSpec, PagedKVSpec
from .attention_biased import distance_rows
from .base import ANY, INIT_EYE, INIT_NORM, INIT_PROJ, INIT_RATE, INIT_SMALL, INIT_TAPS, MATRIX, VECTOR, Mixer, ParamSpec, PositionEncoding, Source


class MaskedAttention(Mixer):
    """``o(softmax(cap(scale * q k^T) + mask) v)`` over a paged cache, ``num_heads`` query heads sharing ``num_kv_heads``
    key/value heads (query head ``h`` reads key/value head ``h // (num_heads // num_kv_heads)``). Options, each off unless asked
    for:

    * ``conv_taps``: a short causal convolution per channel on q, k and v right after their projection (no bias, no
      activation); a request's last ``conv_taps - 1`` projected rows are part of its state;
    * ``qk_norm``: RMS norm of every query and key head with a weight of ``head_dim`` entries shared by the heads, before rotation;
      ``qk_norm="rows"``: of the whole query projection and of the whole key projection at once, with a weight per row of them;
    * ``values_are_keys`` (with ``qk_norm="rows"``, without rotation): there is no value projection, the values are the keys as they
      are before the norm. The cache holds that row ONCE, with one number per token beside it, its reciprocal root mean square:
      the norm's weight is moved to the queries, ``q . (w k rms^-1) = rms^-1 (w q) . k``, and the number multiplies the score;
    * ``bias_far``: a bias ``rel[row(i - j), head]`` (``{prefix}.rel``) is added to the (capped) score, its row chosen by the distance
      (``distance_rows``), the last row from ``bias_far`` on; the number of rows is the checkpoint's;
    * ``position``: a rotary encoding with ``dims`` and ``tables`` (cos, sin of ``[N, dims / 2]``); the first ``dims`` entries of a
      head turn, the rest pass; pairs are ``(i, i + dims/2)``, or neighbours ``(2i, 2i+1)`` when ``interleaved``;
    * ``window`` with ``keep_first``: position i sees ``j <= i`` with ``i - j < window`` or ``j < keep_first``;
    * ``chunk``: position i sees ``j <= i`` with ``floor(i / chunk) == floor(j / chunk)``;
    * ``softcap``: the scaled score s becomes ``softcap * tanh(s / softcap)``;
    * keys and values may differ in size (``head_dim``, ``v_head_dim``);
    * ``talking_heads``: the heads' scaled and capped scores at one (query, key) pair are mixed before mask and softmax,
      ``score'_h = sum_g talk[h, g] score_g`` with ``talk [heads, heads]`` (``{prefix}.talk``);
    * ``sink``: a learned number per head (``{prefix}.sink``) whose exponential joins the softmax's denominator once: it has no key and
      no value and is neither scaled nor capped nor mixed;
    * ``head_gate``: head h's result is multiplied by ``sigmoid(W_g x)_h`` (``{prefix}.g``, one row per head, read from the mixer's input);
    * ``bias``: q, k, v and the output projection have biases (``{prefix}.q.b`` and so on);
    * ``value_position``: a rotary encoding over all ``v_head_dim`` entries of a value: the value of position j turns by j's angles and is
      cached so; every head's result at position i turns back by i's angles, so that the result knows distances (pairs as for q and k);
    * ``log_distance``: ``r1_h ln(1 + r2_h (i - j))`` is taken off head h's scaled score (``{prefix}.r1``, ``{prefix}.r2``);
    * ``scoring = "sigmoid"``: no softmax; a visible key's weight is ``sigmoid(score + pb_h)`` (``{prefix}.pb``), not normalised over keys.

    The three projections are one matrix; norm, rotation and the cache write are one kernel; the mask is never a tensor.
    Pages that neither window nor chunk can reach any more go back to the pool as a request moves on.
    """

    graph_safe = True

    def __init__(self, hidden: int, num_heads: int, num_kv_heads: int, head_dim: int, v_head_dim: int, scale: float, prefix: str,
                 position: Optional[PositionEncoding] = None, interleaved: bool = False, window: Optional[int] = None, keep_first: int = 0,
                 chunk: Optional[int] = None, softcap: Optional[float] = None, conv_taps: int = 0, qk_norm=False, eps: float = 1e-6,
                 talking_heads: bool = False, sink: bool = False, head_gate: bool = False, bias: bool = False,
                 value_position: Optional[PositionEncoding] = None, log_distance: bool = False, scoring: str = "softmax",
                 values_are_keys: bool = False, bias_far: Optional[float] = None, random_rel_rows: int = 16):
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} query heads cannot share {num_kv_heads} key/value heads")
        if keep_first and not window:
            raise ValueError("first tokens can only be kept where a window would pass them")
        if position is not None and position.dims > head_dim:
            raise ValueError(f"{position.dims} rotated dimensions do not fit heads of {head_dim}")
        if conv_taps and not 1 <= conv_taps <= 8:
            raise ValueError(f"a short convolution has 1 to 8 taps, got {conv_taps}")
        self.hidden, self.num_heads, self.num_kv_heads = hidden, num_heads, num_kv_heads
        self.head_dim, self.v_head_dim, self.scale, self.prefix = head_dim, v_head_dim, float(scale), prefix
        self.position, self.interleaved = position, bool(interleaved)
        self.window, self.keep_first, self.chunk = window, int(keep_first), chunk
        self.softcap = float(softcap) if softcap else 0.0
        self.conv_taps, self.qk_norm, self.eps = int(conv_taps), bool(qk_norm), float(eps)
        self.norm_rows = qk_norm == "rows"
        if self.norm_rows and (conv_taps or position is not None or value_position is not None):
            raise ValueError("queries and keys normed as whole projections are not built together with convolutions or rotation")
        self.values_are_keys = bool(values_are_keys)
        if values_are_keys and (not self.norm_rows or v_head_dim != head_dim):
            raise ValueError("values that are the keys need keys normed as a whole projection, and heads of one size")
        if bias_far is not None and (scoring == "sigmoid" or talking_heads):
            raise ValueError("a bias by distance is not built together with sigmoid weights or talking heads")
        self.bias_far, self.random_rel_rows = bias_far, int(random_rel_rows)
        self.rel: Optional[torch.Tensor] = None
        self.rel_rows: Optional[torch.Tensor] = None   # int32 [ceil(bias_far)]: distance -> row of ``rel``
        self.channels = (num_heads + num_kv_heads) * head_dim + (0 if values_are_keys else num_kv_heads * v_head_dim)
        self.talking_heads, self.has_sink, self.head_gate = bool(talking_heads), bool(sink), bool(head_gate)
        if scoring not in ("softmax", "sigmoid"):
            raise ValueError(f"scoring '{scoring}' is not 'softmax' or 'sigmoid'")
        if scoring == "sigmoid" and sink:
            raise ValueError("weights without a softmax have no denominator that a sink could join")
        if value_position is not None and value_position.dims != v_head_dim:
            raise ValueError(f"values of {v_head_dim} entries turn as a whole, not in {value_position.dims} of them")
        if conv_taps and (bias or value_position is not None):
            raise ValueError("biases and turned values are not built together with short convolutions")
        self.has_bias, self.value_position, self.log_distance, self.scoring = bool(bias), value_position, bool(log_distance), scoring
        self.b_qkv: Optional[torch.Tensor] = None
        self.b_o: Optional[torch.Tensor] = None
        self.r1: Optional[torch.Tensor] = None
        self.r2: Optional[torch.Tensor] = None
        self.pb: Optional[torch.Tensor] = None
        self.talk: Optional[torch.Tensor] = None
        self.sink: Optional[torch.Tensor] = None
        self.w_qkv: Optional[torch.Tensor] = None
        self.w_o: Optional[torch.Tensor] = None
        self.conv_w: Optional[torch.Tensor] = None
        self.q_norm: Optional[torch.Tensor] = None
        self.k_norm: Optional[torch.Tensor] = None

    def _rows(self):
        rows = (("q", self.num_heads * self.head_dim), ("k", self.num_kv_heads * self.head_dim))
        return rows if self.values_are_keys else rows + (("v", self.num_kv_heads * self.v_head_dim),)

    def params(self) -> Dict[str, ParamSpec]:
        p, h = self.prefix, self.hidden
        joined = tuple(Source(f"{p}.{n}", (r, h), INIT_PROJ) for n, r in self._rows())
        if self.head_gate:   # the gate's rows ride behind q, k and v in the joined projection
            joined += (Source(f"{p}.g", (self.num_heads, h), INIT_PROJ),)
        out = {"w_qkv": ParamSpec(joined, MATRIX),
               "w_o": ParamSpec((Source(f"{p}.o", (h, self.num_heads * self.v_head_dim), INIT_PROJ),), MATRIX)}
        if self.has_bias:   # (biases are kept in the type of the products they are added to)
            out["b_qkv"] = ParamSpec(tuple(Source(f"{p}.{n}.b", (r,), INIT_SMALL) for n, r in self._rows()), MATRIX)
            out["b_o"] = ParamSpec((Source(f"{p}.o.b", (h,), INIT_SMALL),), MATRIX)
        if self.log_distance:
            out["r1"] = ParamSpec((Source(f"{p}.r1", (self.num_heads,), INIT_RATE),), VECTOR)
            out["r2"] = ParamSpec((Source(f"{p}.r2", (self.num_heads,), INIT_RATE),), VECTOR)
        if self.scoring == "sigmoid":
            out["pb"] = ParamSpec((Source(f"{p}.pb", (self.num_heads,), INIT_SMALL),), VECTOR)
        if self.talking_heads:
            out["talk"] = ParamSpec((Source(f"{p}.talk", (self.num_heads, self.num_heads), INIT_EYE),), VECTOR)
        if self.has_sink:
            out["sink"] = ParamSpec((Source(f"{p}.sink", (self.num_heads,), INIT_SMALL),), VECTOR)
        if self.conv_taps:
            out["conv_w"] = ParamSpec(tuple(Source(f"{p}.{n}.conv", (r, self.conv_taps), INIT_TAPS) for n, r in self._rows()), VECTOR)
        if self.qk_norm:
            heads_q, heads_k = (self.num_heads, self.num_kv_heads) if self.norm_rows else (1, 1)
            out["q_norm"] = ParamSpec((Source(f"{p}.q.norm", (heads_q * self.head_dim,), INIT_NORM),), VECTOR)
            out["k_norm"] = ParamSpec((Source(f"{p}.k.norm", (heads_k * self.head_dim,), INIT_NORM),), VECTOR)
        if self.bias_far is not None:
            out["rel"] = ParamSpec((Source(f"{p}.rel", (ANY, self.num_heads), INIT_SMALL, free=self.random_rel_rows),), VECTOR)
        return out

    def bind(self, tensors) -> None:
        super().bind(tensors)
        pad = -self.w_qkv.shape[0] % 8   # (rows of the product that start on a 16-byte boundary)
        if pad:
            self.w_qkv = torch.cat([self.w_qkv, self.w_qkv.new_zeros((pad, self.w_qkv.shape[1]))]).contiguous()
        if self.b_qkv is not None and self.b_qkv.shape[0] < self.w_qkv.shape[0]:   # (the rows of a gate, and the padding, have no bias)
            self.b_qkv = torch.cat([self.b_qkv, self.b_qkv.new_zeros(self.w_qkv.shape[0] - self.b_qkv.shape[0])]).contiguous()
        if self.rel is not None:
            self.rel = self.rel.contiguous()
            self.rel_rows = torch.tensor(distance_rows(self.rel.shape[0], self.bias_far), dtype=torch.int32, device=self.rel.device)

    def cache_spec(self):
        pages = PagedKVSpec(self.num_kv_heads, self.head_dim, self.window, 0 if self.values_are_keys else self.v_head_dim, self.keep_first, self.chunk,
                            token_scalar=self.values_are_keys)
        if self.conv_taps:
            return (pages, FixedStateSpec((self.conv_taps - 1, self.channels)))
        return pages

    def forward(self, ctx, h, cache, residual):
        K = ctx.K
        if self.norm_rows:
            return self._forward_rows(ctx, h, cache, residual)
        kv, conv_state = cache if self.conv_taps else (cache, None)
        # where nothing else reads the projections, a small batch leaves its float32 sums to the kernel that turns and stores them
        more = {"transient": True} if not (self.head_gate or self.conv_taps) else {}
        if self.has_bias:
            more["bias"] = self.b_qkv
        z = K.linear(h, self.w_qkv, out_dtype=ctx.dtype, **more)
        gate = z if self.head_gate else None   # (its columns lie behind the heads, from ``channels`` on)
        if self.conv_taps:
            z = K.causal_conv(z, 0, self.channels, self.conv_w, None, conv_state.state, ctx)
        cos = sin = None
        dims = 0
        if self.position is not None:
            cos, sin = ctx.position_tables(self.position)
            dims = self.position.dims
        v_turn = ctx.position_tables(self.value_position) if self.value_position is not None else None
        q = K.qk_norm_rope_store(z, self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim, self.q_norm, self.k_norm, self.eps, cos, sin,
                                 dims, self.interleaved, ctx.slot_mapping[kv.group], kv.k, kv.v, ctx.page_size, write_kv=kv.write,
                                 out_dtype=ctx.dtype, **({"v_turn": v_turn} if v_turn is not None else {}))
        more = {}
        if v_turn is not None:
            more["turn"] = (*v_turn, self.interleaved)
        if self.rel is not None:
            more["rel"], more["rel_rows"] = self.rel, self.rel_rows
        if self.log_distance:
            more["log_distance"] = (self.r1, self.r2)
        if self.scoring == "sigmoid":
            more["sigmoid_bias"] = self.pb
        attn = K.attention_ext(q, 0, self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim, kv.k, kv.v, ctx.block_tables[kv.group],
                               ctx.token_seq, ctx.positions, ctx.page_size, self.scale, self.window or 0, ctx.max_context, batch=ctx,
                               keep_first=self.keep_first, chunk=self.chunk or 0, softcap=self.softcap, sink=self.sink, gate=gate,
                               gate_col=self.channels, gate_per_head=True, talk=self.talk, **more)
        if self.has_bias:
            K.linear(attn, self.w_o, add_to=residual, bias=self.b_o)
        else:
            K.linear(attn, self.w_o, add_to=residual)

    def _forward_rows(self, ctx, h, kv, residual):
        """Queries and keys normed as whole projections: one kernel norms both rows of a token, stores its keys (and values) and
        hands the gate's columns on behind the queries, so the projections' sums have no other reader."""
        K = ctx.K
        z = K.linear(h, self.w_qkv, out_dtype=ctx.dtype, transient=True, **({"bias": self.b_qkv} if self.has_bias else {}))
        q = K.qk_rows_norm_store(z, self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim, self.q_norm, self.k_norm, self.eps,
                                 ctx.slot_mapping[kv.group], kv.k, kv.v, kv.scalar, ctx.page_size, gate_cols=self.num_heads if self.head_gate else 0,
                                 write_kv=kv.write, out_dtype=ctx.dtype)
        more = {}
        if self.log_distance:
            more["log_distance"] = (self.r1, self.r2)
        if self.scoring == "sigmoid":
            more["sigmoid_bias"] = self.pb
        attn = K.attention_ext(q, 0, self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim, kv.k, kv.v, ctx.block_tables[kv.group],
                               ctx.token_seq, ctx.positions, ctx.page_size, self.scale, self.window or 0, ctx.max_context, batch=ctx,
                               keep_first=self.keep_first, chunk=self.chunk or 0, softcap=self.softcap, sink=self.sink,
                               gate=q if self.head_gate else None, gate_col=self.num_heads * self.head_dim, gate_per_head=True, talk=self.talk,
                               rel=self.rel, rel_rows=self.rel_rows, key_scale=kv.scalar, **more)
        K.linear(attn, self.w_o, add_to=residual, **({"bias": self.b_o} if self.has_bias else {}))
