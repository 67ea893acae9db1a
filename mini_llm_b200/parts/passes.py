"""How a looped stretch of layers begins each of its passes.

``ConcatEmbeddingInput``: x <- W [x; x_0] + s_t, x_0 the embedded rows and s_t a learned vector of pass t.  The residual
and the embedded rows are 32-bit; on the bfloat16 path each goes into the product as two bfloat16 terms (hi and the
rest), laid side by side as [x hi | x_0 hi | x lo | x_0 lo] against [W | W], so that the residual keeps about 16 bits on
its way through the matrix; the product's epilogue adds s_t and writes 32-bit.
"""
from __future__ import annotations

from .base import ParamSpec, PassInput, register_part


class ConcatEmbeddingInput(PassInput):
    def __init__(self, hidden_size: int, passes: int):
        self.hidden_size, self.passes = int(hidden_size), int(passes)

    def param_specs(self):
        D = self.hidden_size
        return {"weight": ParamSpec((D, 2 * D), "matrix"), "step": ParamSpec((self.passes, D), "vector")}

    def bind(self, params, rt) -> None:
        import torch
        super().bind(params, rt)
        if "weight" in params:
            self.terms = 1 if rt.act_dtype == torch.float32 else 2
            if self.terms == 2:
                self.weight = torch.cat([self.weight, self.weight], 1).contiguous()
            # a row per pass, each on a 16-byte boundary
            D = self.hidden_size
            pad = torch.zeros((self.passes, -(-D // 4) * 4), dtype=torch.float32, device=self.step.device)
            pad[:, :D] = self.step
            self.step = pad

    def forward(self, x, x0, ctx, t):
        ops = self.rt.ops
        T, D = x.shape
        n = 2 * D * self.terms
        cat = ctx.ws.buf("pass_input", T, -(-n // 8) * 8, self.rt.act_dtype)[:, :n]     # rows stay 16-byte aligned
        ops.concat_terms(x, x0, cat, self.terms)
        ops.linear(cat, self.weight, self.step[t, :D], out=x)
        return x


register_part("pass_input", "concat_embedding", ConcatEmbeddingInput)
