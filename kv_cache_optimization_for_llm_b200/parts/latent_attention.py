"""Attention over a cached latent."""

from __future__ import annotations

import torch

from .. import ops
from ..cache.specs import PagedKVSpec
from ..weights.loader import WeightSpec
from .base import Part
from .delta_rule import _stack
from .registry import lookup, register


@register("mixer", "latent_attention")
class LatentAttention(Part):
    """Causal attention whose keys and values come from a low-rank latent, and the queries from one or straight from
    the layer's input.

    ``c_q = rms(W_dq h) * w_dq`` and ``q = W_uq c_q`` (``q_rank`` None: ``q = W_q h``), per head ``dim`` plain dimensions
    followed by ``rot_dim`` rotated ones.  ``W_dkv h`` gives ``kv_rank`` rows that, RMS-normed, are the latent c,
    and ``rot_dim`` more that are one rotated key part shared by all heads.  Per head the plain key
    is ``W_uk c`` and the value ``W_uv c``; score = (q_plain . k_plain + q_rot . k_rot) * scale; query i sees key
    j when ``0 <= i - j < window`` (``window`` None: every key up to i); with ``sink`` (the default) the softmax's denominator also holds ``exp(sink_h)``.  With ``gate`` the heads' results are multiplied
    element by element by ``sigmoid(W_g h)``.  Only [c | rotated part] is cached, one
    row per token (a paged group of one plane).  With ``borrows_latent`` the layer makes no latent of its own and caches
    nothing: its schedule entry names the entry whose rows it attends to, with its own W_uk, W_uv, window and the rest.

    The key up-projection is applied to the queries instead (q_plain^T W_uk,h c = (W_uk,h^T q_plain)^T c),
    attention runs for all heads over the cached rows, and the value up-projection is applied
    to the attended latents; the output projection follows.
    params: hidden_size, heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, sink, gate, borrows_latent, eps,
    position (PartSpec)."""

    @classmethod
    def weight_specs(cls, params):
        h, H, d, r, dv = (params[k] for k in ("hidden_size", "heads", "dim", "rot_dim", "vdim"))
        qr, kr = params["q_rank"], params["kv_rank"]
        specs = {"uk": WeightSpec((H * d, kr)), "uv": WeightSpec((H * dv, kr)), "o": WeightSpec((h, H * dv))}
        if qr:
            specs.update(dq=WeightSpec((qr, h)), dq_norm=WeightSpec((qr,), "vector"), uq=WeightSpec((H * (d + r), qr)))
        else:
            specs["q"] = WeightSpec((H * (d + r), h))
        if not params.get("borrows_latent"):
            specs.update(dkv=WeightSpec((kr + r, h)), dkv_norm=WeightSpec((kr,), "vector"))
        if params.get("sink", True):
            specs["sink"] = WeightSpec((H,), "bias")
        if params.get("gate"):
            specs["g"] = WeightSpec((H * dv, h))
        return specs

    @classmethod
    def kernel_modules(cls, params, dtype):
        return ("latent_attention",) + (("gemm_f32",) if dtype == torch.float32 else ("gemm_bf16", "gemm_bf16_wide"))

    def __init__(self, params, weights, ctx):
        super().__init__(params, weights, ctx)
        self.heads, self.dim, self.rot, self.vdim = (int(params[k]) for k in ("heads", "dim", "rot_dim", "vdim"))
        self.q_rank, self.rank = int(params["q_rank"] or 0), int(params["kv_rank"])
        self.window = int(params["window"]) if params.get("window") else None
        self.borrows = bool(params.get("borrows_latent"))
        self.scale, self.eps = float(params["scale"]), float(params["eps"])
        if self.rank > 512:
            raise ValueError(f"latent_attention: a latent of {self.rank} is refused (up to 512)")
        # What lies behind the latent in a cached row: the rotated part, or, for an odd latent in bfloat16 without one, a
        # zero (the padding behind the latent's rows of the stacked matrix) that makes the row whole words.
        self.behind = self.rot
        if ctx.dtype == torch.bfloat16 and (self.rank + self.rot) % 2:
            if self.rot:
                raise ValueError("latent_attention: in bfloat16 the cached row (kv_rank + rot_dim) must be even")
            self.behind = 1
        names = ["dq" if self.q_rank else "q"] + ([] if self.borrows else ["dkv"]) + (["g"] if params.get("gate") else [])
        self.w_in, starts = _stack([weights[n] for n in names], ctx.dtype)
        at = dict(zip(names, starts))
        self.at_kv, self.at_g = at.get("dkv", 0), at.get("g")
        self.dq_norm, self.dkv_norm = weights.get("dq_norm"), weights.get("dkv_norm")
        self.uq, self.o, self.sink = weights.get("uq"), weights["o"], weights.get("sink")
        # per head: U_k^T [rank, dim] (absorbs the queries) and U_v [vdim, rank] (up-projects the attended latents)
        self.uk_t = weights["uk"].view(self.heads, self.dim, self.rank).transpose(1, 2).contiguous()
        self.uv = weights["uv"].view(self.heads, self.vdim, self.rank).contiguous()
        pos = params.get("position")
        self.position = None
        if pos is not None and self.rot:
            self.position = (ctx.make("position", pos) if ctx.make is not None
                             else lookup("position", pos.kind)(pos.params, {}, ctx))
            if self.position.rotary_dim > self.rot:
                raise ValueError(f"latent_attention: {self.position.rotary_dim} rotary dimensions in a part of {self.rot}")

    def cache_spec(self):
        return PagedKVSpec(1, self.rank + self.behind, self.window, planes=1)

    def activation_widths(self):
        H = self.heads
        return [self.w_in.shape[0], self.q_rank, H * (self.dim + self.rot), 3 * H * self.rank, 2 * H * self.vdim,
                self.o.shape[0]]

    def query_tile_heights(self):
        """Tokens per tile of the tensor-core attention (bfloat16, sizes it takes): the step's batch
        lays the tiles out for it."""
        if self.ctx.dtype != torch.bfloat16 or not ops.LATENT_TC or not ops.latent_attention_tc_supported(self.rank, self.behind):
            return []
        return [ops.latent_tokens_per_tile(self.heads)]

    def forward(self, x, batch, cache):
        d = ops.linear(x, self.w_in)
        cos, sin = self.position.tables() if self.position is not None else (None, None)
        rdims = self.position.rotary_dim if self.position is not None else 0
        table = batch.block_tables[cache.group]
        cq = None
        if self.q_rank or not self.borrows:
            cq = ops.latent_prep(d, self.q_rank, self.at_kv, self.rank, self.behind, rdims, self.dq_norm, self.dkv_norm,
                                 self.eps, cos, sin, batch, table, cache.k, cache.write and not self.borrows)
        q = ops.linear(cq, self.uq) if self.q_rank else d         # without a latent the queries are the product's first columns
        per_head = self.dim + self.rot
        q_abs = ops.head_gemm(q, 0, per_head, self.uk_t)
        lat = ops.latent_attention(q_abs, q, self.dim if self.rot else 0, per_head, cos, sin, rdims, cache.k, table, batch, self.sink,
                                   self.scale, self.heads, self.rank, self.behind, self.window or 0)
        gate = (d, self.at_g) if self.at_g is not None else None
        return ops.linear(ops.head_gemm(lat, 0, self.rank, self.uv, gate), self.o)
