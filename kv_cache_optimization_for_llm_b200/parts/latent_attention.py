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
    to the attended latents; the output projection follows.  Long runs of tokens in bfloat16 (no rotated part, no gate,
    sizes that the prompt kernels for [key | value] rows take) go the other way: the keys and values of all positions that
    the runs see are made once (``ops.latent_step_rows``), and every head attends to rows of its own, which is a multiple
    fewer operations per query and key (dim + vdim against twice the latent) on a faster kernel.  With ``split_decode``
    bfloat16 steps of single tokens deal a request's keys over several blocks and make the products per head on tensor cores:
    faster, but a token's result then differs by rounding between a short portion and a step of its own.
    params: hidden_size, heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, sink, gate, borrows_latent, split_decode,
    eps, position (PartSpec)."""

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
        if dtype == torch.float32:
            return ("latent_attention", "gemm_f32")
        up = ()
        if cls._up_sizes(params, dtype):
            up = ("window_flash_attention",) + (("flash_attention",) if cls._one_size(params) else ())
        return ("latent_attention",) + up + ("gemm_bf16", "gemm_bf16_wide")

    @staticmethod
    def _up_sizes(params, dtype):
        """Whether long runs may make their keys and values: what the prompt kernels over such rows take."""
        return (dtype == torch.bfloat16 and not int(params["rot_dim"]) and not params.get("gate") and int(params["kv_rank"]) % 8 == 0
                and ops.window_flash_attention_supported(int(params["dim"]), int(params["vdim"]), 1, ops.StepRows.PAGE, dtype))

    @staticmethod
    def _one_size(params):
        return int(params["dim"]) == int(params["vdim"]) and int(params["dim"]) in (64, 128)

    def __init__(self, params, weights, ctx):
        super().__init__(params, weights, ctx)
        self.heads, self.dim, self.rot, self.vdim = (int(params[k]) for k in ("heads", "dim", "rot_dim", "vdim"))
        self.q_rank, self.rank = int(params["q_rank"] or 0), int(params["kv_rank"])
        self.window = int(params["window"]) if params.get("window") else None
        self.borrows = bool(params.get("borrows_latent"))
        self.split = bool(params.get("split_decode"))
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
        # and, for long runs, a head's [U_k; U_v] together
        self.ukv = None
        if self._up_sizes(params, ctx.dtype):
            self.ukv = torch.cat([weights["uk"].view(self.heads, self.dim, self.rank), self.uv], dim=1).contiguous()
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
        widths = [self.w_in.shape[0], self.q_rank, H * (self.dim + self.rot), 3 * H * self.rank, 2 * H * self.vdim,
                  self.o.shape[0]]
        if self.ukv is not None:
            widths.append(ops.LATENT_UP_MAX_KEYS * (H * (self.dim + self.vdim) + self.rank))
        return widths

    def query_tile_heights(self):
        """Tokens per tile of the tensor-core attention (bfloat16, sizes it takes): the step's batch
        lays the tiles out for it."""
        heights = []
        if self.ctx.dtype == torch.bfloat16 and ops.LATENT_TC and ops.latent_attention_tc_supported(self.rank, self.behind):
            heights.append(ops.latent_tokens_per_tile(self.heads))
        if self.ukv is not None:
            heights += [ops.rows_tokens_per_tile(1, False), ops.rows_tokens_per_tile(1, True)]
            if self._one_size(self.params):
                heights.append(ops.flash_tokens_per_tile(1, True))
        return heights

    def _over_made_rows(self, q, table, batch, cache):
        """The heads' results [T, heads * vdim] of a step with long runs; ``q`` holds the queries from column 0 on.  Single
        tokens beside the runs attend to the cached rows as in every other step."""
        rows = ops.latent_step_rows(cache.k, table, batch, self.ukv, self.window or 0)
        if self._one_size(self.params) and ops.flash_attention_rows_masked_wanted(batch, self.heads, self.heads, self.dim, self.vdim,
                                                                                  rows.PAGE, self.ctx.dtype, q):
            a = ops.flash_attention_rows_masked(q, None, None, batch, self.heads, self.heads, self.dim, self.scale, sinks=self.sink,
                                                window=self.window or 0, rows=rows)
        else:
            a = ops.window_flash_attention(q, None, None, batch, self.heads, self.heads, self.dim, self.vdim, self.scale,
                                           self.window or 0, 0, False, sinks=self.sink, rows=rows)
        n = batch.num_single
        if n:
            q_abs = ops.head_gemm(q[:n], 0, self.dim, self.uk_t, tensor_cores=self.split)
            lat = ops.latent_attention(q_abs, q[:n], 0, self.dim, None, None, 0, cache.k, table, batch, self.sink, self.scale,
                                       self.heads, self.rank, self.behind, self.window or 0, singles=True, split=self.split)
            a[:n].copy_(ops.head_gemm(lat, 0, self.rank, self.uv, tensor_cores=self.split))
        return a

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
        if self.ukv is not None and ops.latent_up_wanted(batch, self.window or 0):
            return ops.linear(self._over_made_rows(q, table, batch, cache), self.o)
        q_abs = ops.head_gemm(q, 0, per_head, self.uk_t, tensor_cores=self.split)
        lat = ops.latent_attention(q_abs, q, self.dim if self.rot else 0, per_head, cos, sin, rdims, cache.k, table, batch, self.sink,
                                   self.scale, self.heads, self.rank, self.behind, self.window or 0, split=self.split)
        gate = (d, self.at_g) if self.at_g is not None else None
        return ops.linear(ops.head_gemm(lat, 0, self.rank, self.uv, gate, tensor_cores=self.split), self.o)
