"""Token inputs of a layer: what a layer adds to the stream for the tokens themselves.

``table_gate``: a second embedding table has a part of ``dim`` entries for every layer.  With e the layer's part of the token's row and
x the stream behind the layer's feed-forward,
    g = gelu(W_gate x) * e          (the tanh form of gelu)
    y = W_proj g,     x <- x + y / sqrt(mean(y^2) + eps) * w
The norm and the sum are left to whoever reads the stream next (``Pending.normed``), so they cost no kernel.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from . import linear
from .base import TOKEN_INPUTS, TensorSpec, TokenInput
from .feed_forward import GELU_TANH_GATE


@TOKEN_INPUTS.register("table_gate")
class TableGate(TokenInput):
    """Tensor names: ``table`` [vocab, parts * dim], shared by the model's layers; ``<prefix>gate`` [dim, d], ``<prefix>proj`` [d, dim],
    ``<prefix>norm`` [d].  ``index``: which of the ``parts`` parts of the table's rows this layer reads."""

    def __init__(self, prefix: str, table: str, vocab: int, width: int, dim: int, index: int, parts: int, eps: float):
        if not 0 <= index < parts:
            raise ValueError(f"part {index} of a table row of {parts} parts")
        self.prefix, self.table_name, self.vocab, self.width, self.dim = prefix, table, int(vocab), int(width), int(dim)
        self.index, self.parts, self.eps = int(index), int(parts), float(eps)
        self.table = self.w_gate = self.w_proj = self.norm_w = None

    def tensor_specs(self):
        p, d, n = self.prefix, self.width, self.dim
        return [TensorSpec(self.table_name, (self.vocab, self.parts * n), kind="table"), TensorSpec(p + "gate", (n, d)),
                TensorSpec(p + "proj", (d, n)), TensorSpec(p + "norm", (d,), kind="vector", init="norm")]

    def bind(self, tensors):
        p = self.prefix
        self.table, self.w_gate, self.w_proj = tensors[self.table_name], tensors[p + "gate"], tensors[p + "proj"]
        self.norm_w = tensors[p + "norm"].float().contiguous()

    def forward(self, ctx, x):
        z = linear.linear(ctx, x, self.w_gate)
        ops.table_gate(z, ctx.tokens, self.table, self.index * self.dim, z, GELU_TANH_GATE["alpha"], GELU_TANH_GATE["cubic"], err=ctx.err)
        return linear.linear(ctx, z, self.w_proj), self.norm_w, self.eps
