"""An input of the token to every layer: a second embedding table of which each layer reads its own part.

``SideTable`` holds [vocab, parts * dim]; ``TokenSideBranch`` of part i computes, with e the columns [i * dim, (i + 1) * dim)
of the token's row,

    y = W_proj (gelu_tanh(W_gate h) * e)

and leaves the norm and the sum to the layer's ``side_join``.  The gate's product stays 32-bit until it has been multiplied.
"""
from __future__ import annotations

from .base import ParamSpec, TokenSide, TokenTable, register_part


class SideTable(TokenTable):
    def __init__(self, vocab_size: int, parts: int, dim: int):
        self.vocab_size, self.parts, self.dim = int(vocab_size), int(parts), int(dim)

    def param_specs(self):
        return {"table": ParamSpec((self.vocab_size, self.parts * self.dim), "table")}


register_part("token_table", "side", SideTable)


class TokenSideBranch(TokenSide):
    def __init__(self, hidden_size: int, dim: int, part: int):
        self.hidden_size, self.dim, self.part = int(hidden_size), int(dim), int(part)

    def param_specs(self):
        return {"gate_weight": ParamSpec((self.dim, self.hidden_size), "matrix"),
                "proj_weight": ParamSpec((self.hidden_size, self.dim), "matrix")}

    def attach(self, table) -> None:
        if table.dim != self.dim or not (0 <= self.part < table.parts):
            raise ValueError(f"side branch: part {self.part} of {self.dim} columns in a table of {table.parts} x {table.dim}")
        super().attach(table)

    def forward(self, h, ctx, y):
        import torch
        ops = self.rt.ops
        T = h.shape[0]
        mid = ctx.ws.buf("side_mid", T, -(-self.dim // 8) * 8, self.rt.act_dtype)[:, :self.dim]    # rows stay 16-byte aligned
        if T <= ops.SIDE_FEW_TOKENS and self.hidden_size <= ops.SIDE_MAX_WIDTH:      # few tokens: one launch
            ops.token_side_mid(h, self.gate_weight, ctx.token_ids, self.source.table, self.part * self.dim, mid)
        else:
            z = ctx.ws.buf("side_gate", T, -(-self.dim // 8) * 8, torch.float32)[:, :self.dim]
            ops.linear(h, self.gate_weight, None, out=z)
            ops.token_side_gate(z, ctx.token_ids, self.source.table, self.part * self.dim, mid)
        ops.linear(mid, self.proj_weight, None, out=y)


register_part("token_side", "gated", TokenSideBranch)
