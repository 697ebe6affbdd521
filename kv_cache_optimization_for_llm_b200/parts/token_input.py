"""What a layer adds to the residual stream from its tokens alone."""

from __future__ import annotations

import torch

from .. import ops
from ..weights.loader import WeightSpec
from .base import Part
from .registry import register


@register("token_input", "gated_token_rows")
class GatedTokenRows(Part):
    """A row per token and layer, gated by the stream: ``y = W_proj (gelu_tanh(W_gate x) * e)`` with ``e`` the ``dim`` columns
    from ``first`` on of the token's row of a table [vocab_size, table_width] that all layers share (each its own columns).
    The norm behind it and the addition to the stream belong to the block.
    The products' inner sizes are padded to multiples of 8 (16-byte rows), the padding being zeros.
    params: hidden_size, dim, first, vocab_size, table_width."""

    @classmethod
    def weight_specs(cls, params):
        h, n = int(params["hidden_size"]), int(params["dim"])
        return {"table": WeightSpec((int(params["vocab_size"]), int(params["table_width"]))), "gate": WeightSpec((n, h)),
                "proj": WeightSpec((h, n))}

    @classmethod
    def kernel_modules(cls, params, dtype):
        return ("token_input",) + (("gemm_f32",) if dtype == torch.float32 else ("gemm_bf16", "gemm_bf16_wide"))

    def __init__(self, params, weights, ctx):
        super().__init__(params, weights, ctx)
        self.dim, self.first = int(params["dim"]), int(params["first"])
        self.table, self.gate = weights["table"], weights["gate"]
        self.padded = self.dim + -self.dim % 8
        proj = weights["proj"]
        if self.padded != self.dim:
            proj = torch.cat([proj, proj.new_zeros((proj.shape[0], self.padded - self.dim))], dim=1)
        self.proj = proj.contiguous()

    def activation_widths(self):
        return [self.dim, self.padded, self.proj.shape[0]]

    def forward_whole(self, residual, pending, norm, batch):
        """The branch in one launch, the additions in front of it and behind it included: ``pending`` joins the stream, the
        branch reads it, passes the RMS norm ``norm`` and joins it too.  Returns an :class:`ops.Folded`, or None where the step
        or the sizes want the products' own kernels (:meth:`forward`)."""
        if norm.kind != "rmsnorm" or not ops.token_input_step_wanted(residual.shape[0], residual.shape[1], self.dim, self.padded,
                                                                     pending, self.ctx.dtype):
            return None
        return ops.Folded(ops.token_input_step(residual, pending, self.gate, self.proj, norm.weight, norm.eps, self.table, self.first,
                                               batch))

    def forward(self, x, batch):
        a = ops.token_gate(ops.linear(x, self.gate), self.table, self.first, batch, self.padded)
        return ops.linear(a, self.proj)
