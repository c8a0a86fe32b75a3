"""A layer's input that belongs to the token itself.

``gated_token_row``: every token has a row of a second embedding table, one part of ``dim`` numbers for each layer; the
layer gates its part by a projection of the residual stream and projects the result back,

    g = gelu_tanh(W_gate x) * table[token, index * dim : (index + 1) * dim];    x <- x + norm(W_proj g)

The norm and the sum stay pending, so that the next layer's norm (or the head's) takes them in its own launch.  In
steps of few tokens the gate's product, its activation and the gather are one launch.
"""

from __future__ import annotations

import torch

from .. import kernels
from ..matmul import empty_rows, linear
from .base import NormedPending, TensorSpec, TokenInput, make, register


@register("token_input", "gated_token_row")
class GatedTokenRow(TokenInput):
    graph_safe = True

    def __init__(self, hidden_size: int, vocab_size: int, dim: int, index: int, layers: int, norm, names: dict):
        if dim < 1 or not 0 <= index < layers:
            raise ValueError(f"gated_token_row: part {index} of {layers} parts of {dim} numbers")
        self.hidden, self.V, self.dim, self.index, self.layers = int(hidden_size), int(vocab_size), int(dim), int(index), int(layers)
        self.norm = make("norm", norm)
        self.names = dict(names)      # table (all layers ask for the same one), gate, proj
        self.table = self.w_gate = self.w_proj = None

    def children(self):
        return [self.norm]

    def tensor_specs(self):
        n = self.names
        return [TensorSpec(n["table"], (self.V, self.layers * self.dim)), TensorSpec(n["gate"], (self.dim, self.hidden)),
                TensorSpec(n["proj"], (self.hidden, self.dim))]

    def load(self, fetch):
        self.table = fetch(self.names["table"])
        self.w_gate, self.w_proj = fetch(self.names["gate"]).contiguous(), fetch(self.names["proj"])

    def forward(self, x, ctx):
        T = x.shape[0]
        g = empty_rows(T, self.dim, dtype=x.dtype, device=x.device)
        gate = None if T <= kernels.TOKEN_INPUT_SMALL else linear(x, self.w_gate, out_dtype=torch.float32)
        kernels.token_input(x, self.w_gate, self.table, self.index * self.dim, ctx.token_ids, g, ctx.status, gate=gate)
        return NormedPending(linear(g, self.w_proj, out_dtype=torch.float32), self.norm)
