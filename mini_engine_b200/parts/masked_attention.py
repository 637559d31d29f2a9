"""Grouped-query attention with a mask, a sink in the softmax, and choices around scores, rotation and output.

q = W_q h, k = W_k h, v = W_v h, each with a bias when ``bias`` is set (then the output projection has one too, unless
``output_bias`` is False).  Every q
and k head may be RMS-normed: ``qk_norm`` "before" (with a weight of ``dim`` values for q and one for k, shared by the
heads, in front of the rotation) or "after" (no weight, behind the rotation); "row" takes the root mean square over ALL of a
token's q (and of its k), with a weight for every value.  The rotation pairs element i with element
i + rotary_dim / 2 on the first ``rotary_dim`` elements of a head (a ``FrequencyRotary``, whose frequencies may be
rescaled).  ``temperature`` (coef, every): q is multiplied by 1 + coef ln(floor((p + 1) / every) + 1) at position p.
score = q . k * scale, then, with ``softcap`` c, c tanh(score / c), or, with ``distance_bias``, score - r1 ln(1 + r2 (p - j)) with two
learned numbers a head (``r1``, ``r2``).  ``mask``: None (every key j <= p),
("window", size, keep_first): keys with p - j < size or j < keep_first, or ("chunk", size): keys of the query's own
chunk, floor(j / size) = floor(p / size).  The weights are exp(s_j) / (exp(sink_h) + sum exp(s_j)) with a learned number
per head when ``sink`` is set: a term without key or value that is neither scaled nor capped (``sink`` "one": the term is 1,
nothing learned).  ``head_gate``: the mixer's input also makes a gate a head, whose sigmoid scales that head's result.  ``out_scale`` multiplies the
mixer's output (the values carry it, and the output bias).  Keys have ``dim`` elements
and values ``vdim``; the cache is the engine's usual one (pages of keys and of values) with rows of max(dim, vdim)
elements, or with ``pad_rows`` of the next size the tensor-core kernels take (zeros behind keys and values), and it keeps
what the mask can still show: the window (and the first tokens), or the chunk being filled.

Scores, softmax, norms, angles and the rotation are float32; the packed projection returns float32.  The heads can run inside a
mixer that owns the projections (``heads_of``, see ``SideBySide``): ``hosted`` leaves both out.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from .base import DiskSource, KVCacheNeed, Mixer, ParamDecl
from .linear import Linear
from .registry import PartSpec, build_part, register_mixer


class MaskedSinkAttention(Mixer):
    capturable = True

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float, norm_eps: float,
                 position_encoding: Optional[PartSpec | object] = None, qk_norm: Optional[str] = None, bias: bool = False,
                 softcap: Optional[float] = None, mask: Optional[tuple] = None, sink: "bool | str" = True,
                 temperature: Optional[tuple[float, float]] = None, distance_bias: bool = False, out_scale: float = 1.0,
                 pad_rows: bool = False, hosted: bool = False, output_bias: bool = True, head_gate: bool = False):
        super().__init__()
        if sink not in (True, False, "one"):
            raise ValueError(f"sink must be True, False or 'one', got {sink!r}")
        if num_heads < 1 or num_kv_heads < 1 or num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are no multiple of {num_kv_heads} kv heads")
        if qk_norm not in (None, "before", "after", "row"):
            raise ValueError(f"qk_norm must be None, 'before', 'row' or 'after', got {qk_norm!r}")
        if distance_bias and (softcap or sink or (mask is not None and (mask[0] != "window" or (len(mask) > 2 and mask[2])))):
            raise ValueError("a distance bias goes with a plain window at most, without caps and sinks")
        if temperature is not None and not temperature[1] > 0:
            raise ValueError(f"the temperature's step must be positive, got {temperature!r}")
        self.hidden_size, self.num_heads, self.num_kv_heads = hidden_size, num_heads, num_kv_heads
        self.dim, self.vdim = dim, vdim
        self.scale, self.norm_eps = float(scale), float(norm_eps)
        self.qk_norm, self.has_bias, self.has_sink, self.unit_sink = qk_norm, bias, sink is True, sink == "one"
        self.has_output_bias, self.head_gate = bias and output_bias, head_gate
        self.softcap = float(softcap) if softcap else None
        self.temperature = (float(temperature[0]), float(temperature[1])) if temperature is not None else None
        self.distance_bias, self.out_scale, self.pad_rows = bool(distance_bias), float(out_scale), bool(pad_rows)
        self.row = ops.padded_head(max(dim, vdim)) if pad_rows else max(dim, vdim)       # elements of a cache row
        self.q_row = self.row if pad_rows else dim
        self.window, self.keep_first, self.chunk = None, 0, None
        if mask is not None:
            if mask[0] == "window" and int(mask[1]) >= 1:
                self.window, self.keep_first = int(mask[1]), int(mask[2]) if len(mask) > 2 and mask[2] else 0
            elif mask[0] == "chunk" and int(mask[1]) >= 1:
                self.chunk = int(mask[1])
            else:
                raise ValueError(f"mask must be ('window', size, keep_first) or ('chunk', size), got {mask!r}")
        if isinstance(position_encoding, PartSpec):
            position_encoding = build_part("position_encoding", position_encoding)
        self.rope = position_encoding
        if self.rope is not None and (self.rope.layout != "half_split" or not hasattr(self.rope, "freq") or self.rope.rotary_dim > dim):
            raise ValueError("MaskedSinkAttention rotates halves of at most dim elements from a table of frequencies "
                             f"(got layout {self.rope.layout!r}, {self.rope.rotary_dim} of {dim})")
        H, G = num_heads, num_kv_heads
        self.pieces = [("q", H * dim), ("k", G * dim), ("v", G * vdim)]
        self.channels = sum(n for _, n in self.pieces)          # what passes through biases, norms and the rotation
        self.biased = list(self.pieces)
        if head_gate:
            self.pieces.append(("g", H))
        self.heads_width = H * vdim
        self.in_proj = None if hosted else Linear(hidden_size, self.pieces, name="in_proj")
        self.o_proj = None if hosted else Linear(self.heads_width, [("o", hidden_size)], name="o")
        self.defer_output_bias = False        # a block that adds the output bias itself (with the residual sum) sets this
        self._o_bias = None

    def sub_parts(self):
        parts = [("", part) for part in (self.in_proj, self.o_proj) if part is not None]
        if self.rope is not None:
            parts.append(("rot.", self.rope))
        return parts

    def param_decls(self):
        decls = []
        if self.has_bias:
            sources, start = [], 0
            for piece, n in self.biased:
                sources.append(DiskSource(piece + ".b", start, n))
                start += n
            decls.append(ParamDecl("in_bias", (self.channels,), sources=sources, role="vector"))
        if self.has_output_bias:
            decls.append(ParamDecl("o.b", (self.hidden_size,), role="vector"))
        if self.qk_norm == "before":
            decls += [ParamDecl("q.norm", (self.dim,), init="norm", role="vector"), ParamDecl("k.norm", (self.dim,), init="norm", role="vector")]
        if self.qk_norm == "row":
            decls += [ParamDecl("q.norm", (self.num_heads * self.dim,), init="norm", role="vector"),
                      ParamDecl("k.norm", (self.num_kv_heads * self.dim,), init="norm", role="vector")]
        if self.distance_bias:
            decls += [ParamDecl("r1", (self.num_heads,), init="norm", role="vector"), ParamDecl("r2", (self.num_heads,), init="norm", role="vector")]
        if self.has_sink:
            decls.append(ParamDecl("sink", (self.num_heads,), role="vector"))
        return decls

    def finalize(self, dtype, device):
        if self.has_output_bias:
            self._o_bias = (self.p("o.b") * self.out_scale).contiguous() if self.out_scale != 1.0 else self.p("o.b")

    def cache_needs(self):
        return [KVCacheNeed(self.num_kv_heads, self.row, self.window, keep_first=self.keep_first, chunk=self.chunk)]

    def first_weight(self):
        return self.in_proj.weight if self.in_proj is not None else None

    def output_bias(self):
        """The output projection's bias when the caller has asked to add it itself (``defer_output_bias``), else None."""
        return self._o_bias if self.has_output_bias and self.defer_output_bias else None

    def heads_of(self, proj, ctx, call, out) -> None:
        """``proj`` [T, columns of ``pieces``] float32 -> the joined heads in ``out`` [T, heads_width]."""
        H, G, D, V = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        T = proj.shape[0]
        kv = ctx.kv_cache(call.cache_slot)
        q = ctx.buffer("attn_q", (T, H * self.q_row), ctx.act_dtype)
        weighted = self.qk_norm in ("before", "row")
        ops.attn_prep(proj, self.p("in_bias") if self.has_bias else None, self.p("q.norm") if weighted else None,
                      self.p("k.norm") if weighted else None, self.qk_norm, self.norm_eps,
                      self.rope.freq if self.rope is not None and self.rope.rotary_dim else None, ctx.positions,
                      kv.slot_mapping if call.writes_cache else None, q, kv.pool, kv.page_size, H, G, D, V,
                      temperature=self.temperature, v_scale=self.out_scale, magnitude=self.rope.magnitude if self.rope is not None else 1.0)
        gate = proj[:, self.channels:self.channels + H] if self.head_gate else None
        ops.sink_attention(q, gate, out, kv.pool, kv.page_size, kv.block_tables, ctx.attn_meta, H, G, self.q_row, V, self.scale,
                           self.window, self.unit_sink, sinks=self.p("sink") if self.has_sink else None, softcap=self.softcap,
                           keep_first=self.keep_first, chunk=self.chunk, padded=self.pad_rows,
                           bias=(self.p("r1"), self.p("r2")) if self.distance_bias else None, gate_heads=self.head_gate)

    def forward(self, x, ctx, call):
        proj = self.in_proj.forward(x, ctx, "attn_proj", out_dtype=torch.float32)
        out = ctx.buffer("attn_out", (proj.shape[0], self.heads_width), ctx.act_dtype)
        self.heads_of(proj, ctx, call, out)
        y = self.o_proj.forward(out, ctx, "mixer_out")
        if self.has_output_bias and not self.defer_output_bias:
            ops.add_row_vector(y, self._o_bias)
        return y


register_mixer("masked_sink_attention", MaskedSinkAttention)
