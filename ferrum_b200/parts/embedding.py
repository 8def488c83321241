"""Token embedding, learned positions and output head.

Embedding: row t of the table, upcast to the float32 residual stream, no scaling
(crates/model/src/weights.rs:29-51) unless a `scale` is given; a table of learned position
vectors, when the model has one, is added by the same kernel (unscaled).  Output head: logits = W_out x on the wanted rows only;
W_out is its own matrix or, when the file has none, the embedding table
(crates/model/src/llama.rs:28-40,103-111).
"""
from __future__ import annotations

import torch

from ..ops import lib as ops
from .base import CacheNeed, ParamSpec, Part, PositionEncoding, StateNeed
from .linear import STORE_F32, linear


class TokenEmbedding(Part):
    graph_safe = True

    def __init__(self, n_vocab, width, scale=1.0, positions: "LearnedPositions" = None, copies=1, copy_dtype=None,
                 norm=None, restart_dtype=None, bigram: "BigramTable" = None):
        """positions: a `LearnedPositions` part whose vector for a token's position is added to the
        (scaled) embedding; the model lists it as its position encoding, which owns the table.
        copies > 1: the residual rows are [tokens, copies * width], every copy the embedded token (a
        model whose blocks keep several residual streams).  copy_dtype (a 16-bit type): the rows are also left
        in that type in the step's buffer `residual_copy`, for blocks whose sublayers read the residual row
        itself (`PostNormBlock`, which keeps the copy up to date).  norm (an `RMSNorm`, whose parameters are named
        `norm.`): the embedded row passes it before anything else.  restart_dtype: the row (after the norm) is also left in
        that type in the second half of the step's buffer `restart_rows` (see `RestartInput`).  bigram (a `BigramTable`,
        whose parameters are named `bigram.`): a row chosen by the token and the one before it is added to the (scaled) row;
        the token before a portion's first one is part of a request's state, so the embedding then has a `cache_need`."""
        self.n_vocab, self.width, self.scale, self.positions = n_vocab, width, float(scale), positions
        self.copies = int(copies)
        self.norm, self.restart_dtype = norm, restart_dtype
        if norm is not None and (self.scale != 1.0 or positions is not None or self.copies != 1):
            raise ValueError("a normed embedding is neither scaled nor positioned and has one copy")
        self.bigram = bigram
        if bigram is not None and (norm is not None or positions is not None or self.copies != 1):
            raise ValueError("an embedding of token pairs is neither normed nor positioned and has one copy")
        if restart_dtype is not None and norm is None:
            raise ValueError("the restart rows are filled by the embedding's norm")
        self.copy_dtype = copy_dtype if copy_dtype not in (None, torch.float32) else None
        self.w_weight = None

    def param_specs(self):
        return {"weight": ParamSpec((self.n_vocab, self.width))}

    def children(self):
        return [(n, p) for n, p in (("norm.", self.norm), ("bigram.", self.bigram)) if p is not None]

    def cache_need(self):
        return CacheNeed(state=StateNeed((1,), torch.int32)) if self.bigram is not None else CacheNeed()

    def forward(self, ctx, state=None):
        """state: the embedding's own state rows [slots, ...] where its `cache_need` asks for some."""
        h = ctx.buf("hidden", (ctx.token_capacity, self.copies * self.width), torch.float32)
        if self.norm is not None:
            restart = None
            if self.restart_dtype is not None:
                restart = ctx.buf("restart_rows", (ctx.token_capacity, 2 * self.width), self.restart_dtype)[:, self.width:]
            ops.embedding_norm(self.w_weight, ctx.token_ids, self.norm.w_weight, self.norm.eps, h, ctx.err, copy=restart)
            if self.copy_dtype is not None:
                ops.post_norm_add(h, ctx.n_tokens, xc=ctx.buf("residual_copy", (ctx.token_capacity, self.width), self.copy_dtype))
            return h
        if self.bigram is not None:
            b = self.bigram
            ops.embedding_bigram(self.w_weight, b.w_weight, ctx, b.mul_prev, b.mul_cur, state, h, scale=self.scale)
            if self.copy_dtype is not None:
                ops.post_norm_add(h, ctx.n_tokens, xc=ctx.buf("residual_copy", (ctx.token_capacity, self.width), self.copy_dtype))
            return h
        pos = self.positions.w_weight if self.positions is not None else None
        ops.embedding(self.w_weight, ctx.token_ids, h, ctx.err, scale=self.scale, pos_table=pos,
                      positions=ctx.positions if pos is not None else None, copies=self.copies)
        if self.copy_dtype is not None:
            ops.post_norm_add(h, ctx.n_tokens, xc=ctx.buf("residual_copy", (ctx.token_capacity, h.shape[1]), self.copy_dtype))
        return h


class BigramTable(Part):
    """Rows for pairs of neighbouring tokens, found by hashing: a token whose predecessor is `prev` reads row
    (prev * mul_prev + token * mul_cur) mod buckets, a sequence's first token the extra last row."""
    graph_safe = True

    def __init__(self, buckets, width, mul_prev, mul_cur):
        self.buckets, self.width, self.mul_prev, self.mul_cur = int(buckets), width, int(mul_prev), int(mul_cur)
        if self.buckets < 1:
            raise ValueError("a hashed table needs a bucket")
        self.w_weight = None

    def param_specs(self):
        return {"weight": ParamSpec((self.buckets + 1, self.width))}


class LearnedPositions(PositionEncoding):
    """One learned vector per position, added to the embedded token.  The sum happens inside the
    embedding kernel (`TokenEmbedding(positions=...)`); a position past the table raises the step's
    error flag."""
    graph_safe = True

    def __init__(self, n_positions, width):
        self.n_positions, self.width = int(n_positions), width
        self.w_weight = None

    def param_specs(self):
        return {"weight": ParamSpec((self.n_positions, self.width))}


class OutputHead(Part):
    graph_safe = True

    def __init__(self, n_vocab, width, tied_to: TokenEmbedding = None, tied="auto", softcap=0.0):
        """tied: True (no matrix of its own), False (must have one), "auto" (use the file's
        matrix when present, else the embedding: the reference's rule).  softcap c > 0: the logits
        leave as c * tanh(logits / c)."""
        self.n_vocab, self.width, self.tied_to, self.tied = n_vocab, width, tied_to, tied
        self.softcap = float(softcap or 0.0)
        self.w_weight = None

    def param_specs(self):
        if self.tied is True:
            return {}
        return {"weight": ParamSpec((self.n_vocab, self.width), optional=self.tied == "auto")}

    def finalize(self):
        if self.w_weight is None:
            if self.tied_to is None:
                raise ValueError("output head has neither a matrix nor an embedding to share")
            self.w_weight = self.tied_to.w_weight

    def forward(self, x, ctx, n_rows):
        logits = ctx.buf("logits", (ctx.want_capacity, self.n_vocab), torch.float32)
        linear(x, self.w_weight, logits, STORE_F32, ctx, M=n_rows)
        if self.softcap > 0.0:
            ops.softcap(logits, n_rows, self.softcap)
        return logits
