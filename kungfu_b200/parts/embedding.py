"""Token embedding and the output head.

Embedding: x = E[token] * scale, the scale held in 32-bit (reference:
crates/kf-layers/src/basic.rs:16-50; Gemma 2 sets scale = sqrt(width), gemma2.rs:34).
Head: only the rows whose logits are wanted are normalised and multiplied with the
output matrix (the embedding itself when tied), then capped: logits = cap * tanh(logits / cap)
(reference: crates/kf-layers/src/model.rs:155-175, compose.rs:84-99).
"""
from __future__ import annotations

import torch

from .. import ops
from .base import FixedState, Norm, Part


class Embedding(Part):
    def __init__(self, table: torch.Tensor, scale: float = 1.0):
        self.table = table
        self.scale = float(scale)
        self.vocab, self.width = table.shape

    def state_need(self):
        return None

    def forward(self, ctx, cache=None) -> torch.Tensor:
        x = ctx.buf("residual", (ctx.n_rows, self.width), torch.float32)
        ops.embed(ctx.tokens, self.table, self.scale, x)
        return x


class StreamsEmbedding(Embedding):
    """The residual starts as `streams` equal copies of the embedded row: [rows, streams, width]."""

    def __init__(self, table: torch.Tensor, streams: int, scale: float = 1.0):
        super().__init__(table, scale)
        self.streams = int(streams)

    def forward(self, ctx, cache=None) -> torch.Tensor:
        x = ctx.buf("residual", (ctx.n_rows, self.streams, self.width), torch.float32)
        ops.embed(ctx.tokens, self.table, self.scale, x)
        return x


class PairEmbedding(Embedding):
    """x = E[token] * scale + B[row]: a second table read by the token and the one before it, row =
    (previous * mul_prev + token * mul_cur) mod buckets, buckets = B's rows - 1; a sequence's first token reads B's last
    row.  The previous token is kept per request (one integer in a state slot)."""

    def __init__(self, table: torch.Tensor, pair: torch.Tensor, mul_prev: int, mul_cur: int, scale: float = 1.0):
        super().__init__(table, scale)
        self.pair = pair
        self.mul_prev, self.mul_cur = int(mul_prev), int(mul_cur)

    def state_need(self):
        return FixedState((1,), torch.int32)

    def forward(self, ctx, cache=None) -> torch.Tensor:
        x = ctx.buf("residual", (ctx.n_rows, self.width), torch.float32)
        ops.embed_pair(ctx.tokens, self.table, self.pair, self.scale, self.mul_prev, self.mul_cur, cache.state, x, ctx,
                       writes=cache.writes)
        return x


class LmHead(Part):
    def __init__(self, norm: Norm, weight: torch.Tensor, softcap: float = 0.0, scale: float = 1.0):
        """`scale`: the logits are multiplied by it (before the cap).  The product is linear, so the factor goes into the
        norm's 32-bit weights: the rows it multiplies are rounded afterwards, to the same relative precision."""
        self.norm = norm if scale == 1.0 else norm.scaled(scale)
        self.weight = weight            # [vocab, width]; the embedding table itself when tied
        self.softcap = float(softcap)
        self.vocab = weight.shape[0]

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        """32-bit logits [n_wanted, vocab] for the rows `ctx.logit_rows` names."""
        n = ctx.n_logits
        h = self.norm.forward(x, ctx, ctx.act_dtype, rows=ctx.logit_rows)
        logits = ctx.buf("logits", (n, self.vocab), torch.float32)
        ops.linear(h, self.weight, logits, softcap=self.softcap)
        return logits
