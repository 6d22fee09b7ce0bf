"""A further input a layer takes for its tokens, besides the residual.

The model holds a second table of token rows (`TokenSideTable`), one part of `dim` numbers per layer.  A layer's
`TokenSide` reads e, its part of each token's row, and gives

    y = proj (gelu_tanh(gate x) * e)

of the residual x; the block norms y and adds it.  The table is never gathered as a whole: the kernel that applies
the activation to the gate's product fetches each token's part itself (a token id of -1 - r standing for what the
step before drew in its row r, as in the embedding), so that a step launched before its tokens are known to the host
reads the right rows.
"""

from __future__ import annotations

import torch

from .base import ParamSpec, register_part


class TokenSideTable:
    capture_safe = True

    @staticmethod
    def parameters(spec) -> dict[str, ParamSpec]:
        return {"weight": ParamSpec((spec.vocab, spec.parts * spec.dim), "side_table")}

    def __init__(self, spec, tensors, ops, runtime):
        self.spec = spec
        self.table = tensors["weight"]

    def begin(self, ctx) -> None:
        ctx.carried["side_table"] = self.table


class TokenSide:
    capture_safe = True

    @staticmethod
    def parameters(spec) -> dict[str, ParamSpec]:
        return {"gate.weight": ParamSpec((spec.dim, spec.width), "matrix"), "proj.weight": ParamSpec((spec.width, spec.dim), "matrix")}

    def __init__(self, spec, tensors, ops, runtime):
        self.spec, self.ops, self.runtime = spec, ops, runtime
        # zero rows and columns up to a multiple of 16: the product kernels want whole 16-byte rows
        self.padded = -(-spec.dim // 16) * 16
        gate, proj = tensors.pop("gate.weight"), tensors.pop("proj.weight")
        self.w_gate = gate.new_zeros(self.padded, spec.width)
        self.w_gate[: spec.dim] = gate
        self.w_proj = proj.new_zeros(spec.width, self.padded)
        self.w_proj[:, : spec.dim] = proj

    def forward(self, x, ctx):
        spec, rt, ops = self.spec, self.runtime, self.ops
        n = x.shape[0]
        gate = rt.buffer("side_gate", (n, self.padded), torch.float32)
        gate = ops.linear(x, self.w_gate, gate, allow_partials=True)
        fed = rt.buffer("side_fed", (n, self.padded), rt.act_dtype)
        ops.side_gate(gate, ctx.carried["side_table"], ctx.token_ids, ctx.previous_tokens, spec.index * spec.dim, spec.dim, fed)
        delta = rt.buffer("side_delta", (n, spec.width), torch.float32)
        return ops.linear(fed, self.w_proj, delta, allow_partials=True)


register_part("side_table", "token_side_table", TokenSideTable)
register_part("side", "token_side", TokenSide)
