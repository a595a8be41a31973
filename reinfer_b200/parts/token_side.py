"""A part that lets the token's own row come into every layer once more:

    y = W_p ( gelu_tanh(W_g x) * e )        e = the part [index * dim, (index + 1) * dim) of the token's row of a second table

x is the residual stream itself (its bfloat16 rounding in bfloat16 mode), the table holds one row of count * dim numbers a
token for all layers.  What becomes of y is the block's business (`parallel_norms`: an output norm adds it to the stream).

The ids are those the embedding looked up (`ctx.shared`), so a token that the sampler left on the device is found too.  Two
products: the first with activation and row in its epilogue (`ops.gemm_bf16_act`), the second as any output projection.
"""
from __future__ import annotations

from .. import ops
from ..weights.params import ParamSpec
from .base import FeedForward, register_part
from .embedding import TOKEN_IDS_KEY
from .ffn import activated
from .linear import matmul_into_residual
from .norm import RoundedRows


class TokenSide(FeedForward):
    def __init__(self, hidden: int, dim: int, vocab: int, index: int, count: int, table_name: str = "side.embed",
                 names=("gate", "proj"), activation: str = "gelu_tanh"):
        """index, count: which of the table's `count` parts this layer reads.  The names are whole tensor names where the
        part's prefix is empty: the table is shared by the layers."""
        self.hidden, self.dim, self.vocab, self.index, self.count = int(hidden), int(dim), int(vocab), int(index), int(count)
        if not 0 <= self.index < self.count or self.dim <= 0:
            raise ValueError(f"token side: part {index} of {count}, {dim} numbers each")
        if activation not in ops.ACTS:
            raise ValueError(f"token side: activation {activation!r} (known: {sorted(ops.ACTS)})")
        self.activation, self.table_name = activation, str(table_name)
        self.gate_name, self.proj_name = names
        self.w_gate = self.w_proj = self.rows = self.reads = None

    def param_specs(self):
        return {self.table_name: ParamSpec((self.vocab, self.count * self.dim), init="table"),
                self.gate_name: ParamSpec((self.dim, self.hidden)), self.proj_name: ParamSpec((self.hidden, self.dim))}

    def bind(self, t):
        self.w_gate, self.w_proj = t[self.gate_name], t[self.proj_name]
        self.rows = t[self.table_name][:, self.index * self.dim:(self.index + 1) * self.dim]     # a view: the table stays one tensor
        self.reads = RoundedRows(self.hidden, self.w_gate.device)       # what a product in front may leave for this part

    def forward(self, ctx, xn, residual):
        g = activated(ctx, xn, self.w_gate, self.activation, mul=(self.rows, ctx.shared[TOKEN_IDS_KEY]))
        return matmul_into_residual(ctx, g, self.w_proj, residual)


register_part("ffn", "token_side", TokenSide)
