"""What a token's identity adds to every layer: a row of its own, opened by the stream.

``e`` is the layer's slice of the token's row in one table for all layers, columns ``index * dim .. (index + 1) * dim - 1``;
``y = W_proj (gelu_tanh(W_gate x) * e)`` with x the 32-bit stream itself, and ``x <- x + y / sqrt(mean(y^2) + eps) * w``.

The last step is one pass over the stream, and if the sublayer that reads the stream next has a norm over whole rows, that
norm is in the pass too (``ctx.next_norm``; the normed rows wait in ``ctx.normed_ahead`` for the arrangement that
would have made them).  A step of few tokens computes the gate's product, its gelu and the row in one kernel.
"""

from __future__ import annotations

import torch

from .base import Part, register_part
from .spec import WeightSpec


class TokenSideInput(Part):
    graph_safe = True

    def __init__(self, prefix, vocab_size: int, width: int, dim: int, index: int, n_layers: int, eps: float,
                 table_name: str = "side.embed", gate_name: str = "side.gate", proj_name: str = "side.proj", norm_name: str = "side.norm"):
        super().__init__(prefix)
        self.vocab_size, self.width, self.dim, self.index, self.n_layers = int(vocab_size), int(width), int(dim), int(index), int(n_layers)
        self.eps, self.table_name = float(eps), table_name
        self.names = dict(gate=gate_name, proj=proj_name, norm=norm_name)
        if self.dim < 1 or not 0 <= self.index < self.n_layers:
            raise ValueError(f"{prefix}: slice {self.index} of {self.n_layers}, {self.dim} entries each")

    def weight_specs(self):
        n = self.names
        return [WeightSpec(self.table_name, (self.vocab_size, self.n_layers * self.dim), role="table", init="table"),
                WeightSpec(self.full_name(n["gate"]), (self.dim, self.width)),
                WeightSpec(self.full_name(n["proj"]), (self.width, self.dim)),
                WeightSpec(self.full_name(n["norm"]), (self.width,), role="vector", init="gain")]

    def forward(self, ctx, hidden):
        k, n, names = ctx.kernels, hidden.shape[0], self.names
        opened = ctx.buffer("token_side", (n, self.dim), ctx.act_dtype)
        k.token_gate(ctx, opened, hidden, self.w(names["gate"]), self.weights[self.table_name], self.index * self.dim)
        y = ctx.buffer("token_side_out", (n, self.width), torch.float32)
        k.linear(ctx, y, opened, self.w(names["proj"]))
        ahead = getattr(ctx, "next_norm", None)
        if ahead is not None and getattr(ahead, "whole_row", False):
            normed = ctx.buffer("norm_1", (n, self.width), ctx.act_dtype)
            k.add_normed_norm(ctx, hidden, y, self.w(names["norm"]), self.eps, normed, ahead.w(ahead.name), ahead.eps)
            ctx.normed_ahead = (ahead, normed)
        else:
            k.add_normed_cast(hidden, y, self.w(names["norm"]), self.eps)


register_part("token_side_input", TokenSideInput)
