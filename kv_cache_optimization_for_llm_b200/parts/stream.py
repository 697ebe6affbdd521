"""Parts that stand in the schedule in front of a layer and change what is pending on the
residual stream."""

from __future__ import annotations

import torch

from .. import ops
from ..weights.loader import WeightSpec
from .base import Part
from .registry import register


@register("stream", "pass_start")
class PassStart(Part):
    """The start of pass ``index`` through a run of layers that repeats with the same weights:
    row ``index`` of a learned table [passes, size] joins the stream, and so does, when
    ``add_embedding`` is set, the embedding's output once more.  Nothing is launched here: both
    are added to what is pending, and the next norm sums everything in its own kernel.
    params: size, passes, index, add_embedding."""

    @classmethod
    def weight_specs(cls, params):
        return {"steps": WeightSpec((params["passes"], params["size"]), "bias")}

    @classmethod
    def kernel_modules(cls, params, dtype):
        return ("rowwise",)

    def __init__(self, params, weights, ctx):
        super().__init__(params, weights, ctx)
        index = int(params["index"])
        if not 0 <= index < int(params["passes"]):
            raise ValueError(f"pass_start: pass {index} of {params['passes']}")
        self.vector = weights["steps"][index].contiguous()
        self.needs_embedding = bool(params.get("add_embedding"))

    def forward(self, residual, delta, embedded):
        if delta is None:
            pending = ops.PendingSum()
        elif isinstance(delta, ops.PendingSum):
            pending = delta
        elif isinstance(delta, ops.Folded):
            pending = ops.PendingSum()      # that branch has added its output to the residual itself
        elif isinstance(delta, ops.PostNormed):
            pending = ops.PendingSum((delta.materialize(),))
        else:
            pending = ops.PendingSum((delta,))
        return pending.plus(rows=embedded if self.needs_embedding else None, vector=self.vector)


@register("stream", "pass_entry")
class PassEntry(Part):
    """The start of pass ``index`` through a run of layers that repeats with the same weights: the stream becomes
    ``W [x; x0] + v_index``, a product over the stream x and the embedding's output x0 side by side (``in``: [size,
    2 size], x first), plus row ``index`` of a learned table [passes, size].

    ``W [x; x0] = W_x x + W_0 x0``, and the second half is the same in every pass: it is made once a step
    (``from_embedding``, one small product with float32 result).  A pass then costs the stream's copy in the compute
    type and one product with float32 result; that result takes the stream's place, and the second half and the vector
    join it, in the kernel of the next norm.
    params: size, passes, index."""

    @classmethod
    def weight_specs(cls, params):
        n = int(params["size"])
        return {"in": WeightSpec((n, 2 * n)), "steps": WeightSpec((int(params["passes"]), n), "bias")}

    @classmethod
    def kernel_modules(cls, params, dtype):
        return ("rowwise",) + (("gemm_f32",) if dtype == torch.float32 else ("gemm_bf16", "gemm_bf16_wide"))

    def __init__(self, params, weights, ctx):
        super().__init__(params, weights, ctx)
        index, n = int(params["index"]), int(params["size"])
        if not 0 <= index < int(params["passes"]):
            raise ValueError(f"pass_entry: pass {index} of {params['passes']}")
        self.vector = weights["steps"][index].contiguous()
        # the passes share their matrix: its halves are laid out once
        self.embedding_key = ("pass_entry", weights["in"].data_ptr())
        if self.embedding_key not in ctx.shared:
            ctx.shared[self.embedding_key] = (weights["in"][:, :n].contiguous(), weights["in"][:, n:].contiguous())
        self.w_x, self.w_0 = ctx.shared[self.embedding_key]

    def from_embedding(self, residual):
        """What the embedding's output contributes to every pass: float32 [T, size]."""
        return ops.linear(ops.add_norm(residual, None, "copy", None, 0.0, self.ctx.dtype), self.w_0, out_dtype=torch.float32)

    def forward(self, residual, delta, embedded):
        if isinstance(delta, ops.PendingSum):
            ops.join_norm(residual, delta, None, None, 0.0, self.ctx.dtype, compute_dtype=self.ctx.dtype)
            delta = None
        elif isinstance(delta, ops.Folded):
            delta = None        # that branch has added its output to the residual itself
        x = ops.add_norm(residual, delta, "copy", None, 0.0, self.ctx.dtype)
        return ops.PendingSum(base=ops.linear(x, self.w_x, out_dtype=torch.float32), rows=embedded, vector=self.vector)
