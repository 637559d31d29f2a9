"""Grouped-query attention with two maps a head, whose results are subtracted from one another.

q = W_q h has ``num_heads`` heads of two maps of ``dim`` elements side by side, k = W_k h ``num_kv_heads`` such heads, v = W_v h
heads of ``vdim`` elements.  Each map of q and k is rotated by itself (element i with element i + rotary_dim / 2 on its first
``rotary_dim`` elements).  Each map is a causal softmax attention of its own, score = q . k * scale, over the same values; with
their results a_1, a_2 and

    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff       (one number, from four learned vectors of ``dim`` values)
    o = a_1 - lambda a_2,   o <- o / sqrt(mean(o^2) + eps) * (1 - diff)      (per head, over its ``vdim`` values)

the joined heads pass W_o.

The cache holds a key head as ONE row, its two maps side by side, beside the row of its value; a query map is a query row of the
same width with zeros in the other map's place, so the two maps are two query heads of one group that share every key and value
they load, on the engine's usual attention kernels (rows are filled with zeros up to the next size the tensor-core kernels take).
Scores, softmax, angles, rotation, the difference and its norm are float32; the packed projection returns float32.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from .base import KVCacheNeed, Mixer, ParamDecl
from .linear import Linear
from .registry import PartSpec, build_part, register_mixer


class DifferentialAttention(Mixer):
    capturable = True

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float, diff: float,
                 norm_eps: float, position_encoding: Optional[PartSpec | object] = None, window: Optional[int] = None):
        super().__init__()
        if num_heads < 1 or num_kv_heads < 1 or num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are no multiple of {num_kv_heads} kv heads")
        if min(dim, vdim) < 1:
            raise ValueError("DifferentialAttention: sizes must be positive")
        self.hidden_size, self.num_heads, self.num_kv_heads, self.dim, self.vdim = hidden_size, num_heads, num_kv_heads, dim, vdim
        self.scale, self.diff, self.norm_eps, self.window = float(scale), float(diff), float(norm_eps), window
        if isinstance(position_encoding, PartSpec):
            position_encoding = build_part("position_encoding", position_encoding)
        self.rope = position_encoding
        if self.rope is not None and (self.rope.layout != "half_split" or not hasattr(self.rope, "freq") or self.rope.rotary_dim > dim):
            raise ValueError("DifferentialAttention rotates halves of at most dim elements from a table of frequencies "
                             f"(got layout {self.rope.layout!r}, {self.rope.rotary_dim} of {dim})")
        self.row = ops.padded_head(max(2 * dim, vdim))
        self.in_proj = Linear(hidden_size, [("q", num_heads * 2 * dim), ("k", num_kv_heads * 2 * dim), ("v", num_kv_heads * vdim)], name="in_proj")
        self.o_proj = Linear(num_heads * vdim, [("o", hidden_size)], name="o")
        self.lam = None

    def sub_parts(self):
        parts = [("", self.in_proj), ("", self.o_proj)]
        if self.rope is not None:
            parts.append(("rot.", self.rope))
        return parts

    def param_decls(self):
        return [ParamDecl(n, (self.dim,), role="vector") for n in ("lq1", "lk1", "lq2", "lk2")]

    def finalize(self, dtype, device):
        v = {n: self.p(n).double() for n in ("lq1", "lk1", "lq2", "lk2")}
        self.lam = float(torch.exp((v["lq1"] * v["lk1"]).sum()) - torch.exp((v["lq2"] * v["lk2"]).sum())) + self.diff

    def cache_needs(self):
        return [KVCacheNeed(self.num_kv_heads, self.row, self.window)]

    def first_weight(self):
        return self.in_proj.weight

    def forward(self, x, ctx, call):
        H, G, D, V = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        proj = self.in_proj.forward(x, ctx, "attn_proj", out_dtype=torch.float32)
        T = proj.shape[0]
        kv = ctx.kv_cache(call.cache_slot)
        q = ctx.buffer("attn_q", (T, 2 * H * self.row), ctx.act_dtype)
        rotated = self.rope is not None and self.rope.rotary_dim > 0
        ops.attn_prep(proj, None, None, None, None, self.norm_eps, self.rope.freq if rotated else None, ctx.positions,
                      kv.slot_mapping if call.writes_cache else None, q, kv.pool, kv.page_size, H, G, D, V, maps=2)
        out = ctx.buffer("attn_out", (T, H * V), ctx.act_dtype)
        ops.sink_attention(q, None, out, kv.pool, kv.page_size, kv.block_tables, ctx.attn_meta, 2 * H, G, self.row, V, self.scale,
                           self.window, False, padded=True, pairs=(self.lam, 1.0 - self.diff, self.norm_eps))
        return self.o_proj.forward(out, ctx, "mixer_out")


register_mixer("differential_attention", DifferentialAttention)
