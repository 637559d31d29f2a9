"""Mixers that read the same input side by side and whose outputs are added.

``mixers`` is a list of (prefix of its tensors, mixer kind and arguments).  The inner mixers must be of kinds that can run their heads
alone (``pieces``: the rows their input projection is made of; ``heads_width``: the columns of their joined heads;
``heads_of(proj, ctx, call, out)``) and are built ``hosted``, without projections of their own: this mixer packs all input
projections into ONE product and all output projections into one, whose input is the joined heads of all mixers side by side, so
that their sum costs nothing.  ``output_norms`` = {"names": [a weight's name for every mixer], "eps", "mean": bool} instead: every
mixer's output passes an RMS norm of its own over the model width, with a plain weight, before the sum (or, with ``mean``, the mean);
then every mixer has an output product of its own and the result is a ``PendingSum`` of ``PendingTerm``s, so that the norms run in the
kernel that adds to the stream.  A factor on a mixer's output is that mixer's ``out_scale``.  Output biases (``output_bias()`` of an
inner mixer) are added by this mixer, or by the block that runs it (``defer_output_bias``)."""
from __future__ import annotations

from typing import Optional, Sequence

import torch

from .. import ops
from .base import Mixer, ParamDecl, PendingSum, PendingTerm
from .linear import Linear
from .registry import PartSpec, build_part, register_mixer


class SideBySide(Mixer):
    def __init__(self, hidden_size: int, mixers: Sequence[tuple[str, PartSpec]], output_norms: Optional[dict] = None):
        super().__init__()
        self.hidden_size = hidden_size
        self.prefixes = [p for p, _ in mixers]
        self.mixers = [build_part("mixer", PartSpec(s.kind, {**s.args, "hosted": True})) for _, s in mixers]
        self.capturable = all(m.capturable for m in self.mixers)
        in_pieces, out_pieces, self.columns, self.out_columns, col, out_col = [], [], [], [], 0, 0
        for prefix, m in zip(self.prefixes, self.mixers):
            if not hasattr(m, "heads_of"):
                raise ValueError(f"{type(m).__name__} cannot run beside another mixer (it has no heads_of)")
            in_pieces += [(prefix + name, rows) for name, rows in m.pieces]
            width = sum(rows for _, rows in m.pieces)
            self.columns.append((col, col + width))
            out_pieces.append((prefix + "o", m.heads_width))
            self.out_columns.append((out_col, out_col + m.heads_width))
            col, out_col = col + width, out_col + m.heads_width
            if hasattr(m, "defer_output_bias"):
                m.defer_output_bias = True
        self.width = out_col
        self.in_proj = Linear(hidden_size, in_pieces, name="in_proj")
        self.output_norms, self.o_projs, self._norm_weights = None, [], []
        if output_norms is None:
            self.o_proj = Linear(self.width, name="o_proj", input_pieces=out_pieces, out_features=hidden_size)
        else:
            self.o_proj = None
            self.output_norms = dict(output_norms)
            if len(self.output_norms["names"]) != len(self.mixers):
                raise ValueError("SideBySide: every mixer needs the name of its output norm's weight")
            self.o_projs = [Linear(m.heads_width, [(name, hidden_size)], name=name) for m, (name, _) in zip(self.mixers, out_pieces)]
        self.defer_output_bias = False        # a block that adds the output biases itself (with the residual sum) sets this
        self._bias = None

    def sub_parts(self):
        projs = [self.o_proj] if self.o_proj is not None else self.o_projs
        return [("", self.in_proj)] + [("", o) for o in projs] + list(zip(self.prefixes, self.mixers))

    def param_decls(self):
        names = self.output_norms["names"] if self.output_norms else []
        return [ParamDecl(n, (self.hidden_size,), init="norm", role="vector") for n in names]

    def finalize(self, dtype, device):
        if self.output_norms:
            factor = 1.0 / len(self.mixers) if self.output_norms.get("mean") else 1.0
            self._norm_weights = [(self.p(n) * factor).contiguous() for n in self.output_norms["names"]]

    def cache_needs(self):
        return [need for m in self.mixers for need in m.cache_needs()]

    def first_weight(self):
        return self.in_proj.weight

    def _summed_bias(self):
        if self._bias is None:
            found = [b for m in self.mixers if hasattr(m, "output_bias") and (b := m.output_bias()) is not None]
            self._bias = sum(found[1:], found[0]).contiguous() if found else False
        return None if self._bias is False else self._bias

    def output_bias(self):
        """The sum of the output biases when the caller has asked to add it itself (``defer_output_bias``), else None."""
        return self._summed_bias() if self.defer_output_bias else None

    def forward(self, x, ctx, call):
        proj = self.in_proj.forward(x, ctx, "side_by_side_proj", out_dtype=torch.float32)
        if self.output_norms:
            if self._summed_bias() is not None:
                raise ValueError("SideBySide: output biases and output norms do not go together")
            terms = []
            for i, (m, (a, b), o) in enumerate(zip(self.mixers, self.columns, self.o_projs)):
                heads = ctx.buffer(f"side_by_side_heads{i}", (proj.shape[0], m.heads_width), ctx.act_dtype)
                m.heads_of(proj[:, a:b], ctx, call, heads)
                terms.append(PendingTerm(o.forward(heads, ctx, f"mixer_out{i}"), self._norm_weights[i], float(self.output_norms["eps"])))
            return PendingSum(terms)
        heads = ctx.buffer("side_by_side_heads", (proj.shape[0], self.width), ctx.act_dtype)
        for m, (a, b), (c, d) in zip(self.mixers, self.columns, self.out_columns):
            m.heads_of(proj[:, a:b], ctx, call, heads[:, c:d])
        y = self.o_proj.forward(heads, ctx, "mixer_out")
        if not self.defer_output_bias and self._summed_bias() is not None:
            ops.add_row_vector(y, self._bias)
        return y


register_mixer("side_by_side", SideBySide)
