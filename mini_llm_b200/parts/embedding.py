"""Token embedding, learned absolute positions, and the output head.

``hidden[t] = wte[id_t] + wpe[pos_t]`` with ``pos_t`` the token's absolute
position in its request (engine/src/embedding.c:9-15; with an offset for
cached tokens, engine/src/embedding.cu:21-26,100-103).  The head multiplies
the normed rows whose logits are wanted with the token table itself, without
bias (engine/src/gpt2.c:245-256); the reference keeps a transposed copy of
the table for this (engine/src/gpt2_gpu.cu:32-48), here the one [vocab, width]
table serves the gather and the product.  ``scale`` multiplies the gathered rows (in 32-bit), not the head's.
"""

from __future__ import annotations

import torch

from .base import Embedding, Head, PositionEncoding, register_part
from .spec import FixedState, WeightSpec


class TokenEmbedding(Embedding):
    graph_safe = True
    def __init__(self, prefix, vocab_size: int, width: int, name: str = "wte.weight", scale: float = 1.0):
        super().__init__(prefix)
        self.vocab_size, self.width, self.name, self.scale = int(vocab_size), int(width), name, float(scale)

    def weight_specs(self):
        return [WeightSpec(self.full_name(self.name), (self.vocab_size, self.width), role="table", init="table")]

    def forward(self, ctx, position=None, cache=None):
        hidden = ctx.buffer("hidden", (ctx.n_tokens, self.width), torch.float32)
        table = position.additive_table() if position is not None else None
        ctx.kernels.embed(hidden, ctx.token_ids, ctx.positions, self.w(self.name), table, self.scale)
        if position is not None and table is None:
            position.add_to_hidden(ctx, hidden)
        return hidden


class PairedTokenEmbedding(TokenEmbedding):
    """The token's row plus a row for the pair of it and the token before it: row
    ``(previous * mul_prev + token * mul_cur) mod buckets`` of a table of ``buckets + 1`` rows, the last of which is for a
    sequence's first token.  A request's last token is its state."""

    def __init__(self, prefix, vocab_size: int, width: int, buckets: int, mul_prev: int, mul_cur: int, name: str = "wte.weight",
                 pair_name: str = "bigram", scale: float = 1.0):
        super().__init__(prefix, vocab_size, width, name, scale)
        self.buckets, self.mul_prev, self.mul_cur, self.pair_name = int(buckets), int(mul_prev), int(mul_cur), pair_name
        if self.buckets < 1 or min(self.mul_prev, self.mul_cur) < 0:
            raise ValueError(f"{self.full_name(pair_name)}: a positive number of buckets and factors that are not negative")

    def weight_specs(self):
        return super().weight_specs() + [WeightSpec(self.full_name(self.pair_name), (self.buckets + 1, self.width), role="table", init="table")]

    def cache_need(self):
        return FixedState((1,), "int32")

    def forward(self, ctx, position=None, cache=None):
        hidden = ctx.buffer("hidden", (ctx.n_tokens, self.width), torch.float32)
        ctx.kernels.pair_embed(ctx, hidden, self.w(self.name), self.w(self.pair_name), cache.state.view(-1), self.buckets, self.mul_prev,
                               self.mul_cur, self.scale)
        if position is not None:
            position.add_to_hidden(ctx, hidden)
        return hidden


class LearnedPositions(PositionEncoding):
    """A table row per absolute position, added to the embedded token."""
    graph_safe = True

    def __init__(self, prefix, max_positions: int, width: int, name: str = "wpe.weight"):
        super().__init__(prefix)
        self.max_positions, self.width, self.name = int(max_positions), int(width), name

    def weight_specs(self):
        return [WeightSpec(self.full_name(self.name), (self.max_positions, self.width), role="table", init="table")]

    def additive_table(self):
        return self.w(self.name)

    def add_to_hidden(self, ctx, hidden):
        ctx.kernels.add_position_rows(hidden, ctx.positions, self.w(self.name))


class LinearHead(Head):
    """logits = x W^T, W [vocab, width].  ``weight_name`` may be the token
    table's name (tied head): the loader then shares the one tensor.  With ``softcap`` the logits are
    then capped, ``cap * tanh(logits / cap)``."""
    graph_safe = True

    def __init__(self, prefix, vocab_size: int, width: int, weight_name: str = "lm_head.weight", softcap: float | None = None):
        super().__init__(prefix)
        self.vocab_size, self.width, self.weight_name = int(vocab_size), int(width), weight_name
        self.softcap = float(softcap) if softcap else None      # logits <- cap * tanh(logits / cap)

    def weight_specs(self):
        return [WeightSpec(self.full_name(self.weight_name), (self.vocab_size, self.width), role="table", init="table")]

    accepts_deferred_norm = True

    def forward(self, ctx, x):
        logits = ctx.buffer("logits", (x.shape[0], self.vocab_size), torch.float32)
        ctx.kernels.linear(ctx, logits, x, self.w(self.weight_name), None)
        if self.softcap is not None:
            ctx.kernels.softcap(logits, self.softcap)
        return logits


register_part("token_embedding", TokenEmbedding)
register_part("paired_token_embedding", PairedTokenEmbedding)
register_part("learned_positions", LearnedPositions)
register_part("linear_head", LinearHead)
