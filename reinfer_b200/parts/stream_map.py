"""A linear map of the residual stream beside the embedding's output, x <- W [x; x0] with W [hidden, 2 hidden] (x first), for
block `stream_map`: a stretch of layers that runs several times reads the embedding anew before every pass.

W is used as its two halves, x <- W_1 x + W_2 x0.  The second term is the same in every pass: it is formed once a step in
32-bit and copied into the stream, and the first product adds to it - a pass then reads half of W, and the product may do
what any output projection does (make the next norm's rows, or leave partial sums to it).  In bfloat16 the products read
the stream's and the embedding's roundings; sums and stream are 32-bit.
"""
from __future__ import annotations

import torch

from ..weights.params import ParamSpec
from .base import FeedForward, register_part
from .embedding import OUTPUT_KEY
from .linear import matmul, matmul_into_residual
from .norm import RoundedRows


class StreamRecall(FeedForward):
    def __init__(self, hidden: int, weight_name: str = "weight"):
        """weight_name: the local name of the matrix ("" where the part's prefix is the whole name)."""
        self.hidden, self.weight_name = int(hidden), str(weight_name)
        self.w_x = self.w_first = self.reads = None

    def param_specs(self):
        return {self.weight_name: ParamSpec((self.hidden, 2 * self.hidden))}

    def bind(self, t):
        w = t[self.weight_name]
        self.w_x, self.w_first = w[:, :self.hidden].contiguous(), w[:, self.hidden:].contiguous()
        self.reads = RoundedRows(self.hidden, w.device)         # what the block in front may leave for this part

    def forward(self, ctx, rows, x):
        """rows: x as the product reads it (the stream itself, or its rounding).  x is replaced."""
        key = ("stream_recall", id(self))
        first = ctx.shared.get(key)
        if first is None:
            first = ctx.shared[key] = matmul(ctx, ctx.shared[OUTPUT_KEY], self.w_first, out_dtype=torch.float32)
        if rows is x:
            rows = x.clone()                                    # (32-bit: the product's input and its sum may not be one tensor)
        x.copy_(first)
        return matmul_into_residual(ctx, rows, self.w_x, x)


register_part("ffn", "stream_recall", StreamRecall)
