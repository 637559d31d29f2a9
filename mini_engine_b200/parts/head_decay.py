"""Linear attention whose state decays by one number a head: a constant (retention) or one that the input makes (Mamba-2); a state slot
per request.

Per head: S_t = a_t S_(t-1) + g_t k_t v_t^T, o_t = S_t^T q_t, S (``dim`` x ``vdim``) starting at zero.  States, decays, their logarithms
and everything of the recurrence are float32; what enters it (the projections, the short convolution with its activation) is in the
working dtype.  Both run the kernels of csrc/head_decay.cu, which also know keys and queries that neighbouring heads share.
"""
from __future__ import annotations

import math
from typing import Sequence

import torch

from .. import ops
from .base import Mixer, ParamDecl, StateNeed
from .linear import Linear
from .registry import register_mixer


def _workspaces(ctx, heads: int, dim: int, vdim: int) -> dict:
    runs = ops.head_decay_chunk_count(ctx.attn_meta)
    if not runs:
        return {}
    return {"chunk_states": ctx.buffer("head_decay_states", (runs, heads, dim, vdim), torch.float32),
            "run_numbers": ctx.buffer("head_decay_run_numbers", (runs, heads, ops.HEAD_DECAY_RUN), torch.float32)}


class Retention(Mixer):
    """q = W_q x, k = W_k x * dim^-1/2, v = W_v x; a_t is the head's entry of ``decay``, the same for every token, and g_t = 1.  An RMS norm
    without a weight brings each head's o to unit size, silu(W_g x) gates the joined heads, and W_o takes them back to the stream's width."""
    capturable = True

    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, decay: Sequence[float], norm_eps: float):
        super().__init__()
        if min(num_heads, dim, vdim) < 1:
            raise ValueError("Retention: sizes must be positive")
        if len(decay) != num_heads or not all(0.0 < d <= 1.0 for d in decay):
            raise ValueError(f"Retention: every one of the {num_heads} heads needs a decay above 0 and up to 1, got {list(decay)}")
        self.hidden_size, self.num_heads, self.dim, self.vdim = hidden_size, num_heads, dim, vdim
        self.decay, self.norm_eps = [float(d) for d in decay], float(norm_eps)
        H = num_heads
        self.in_proj = Linear(hidden_size, [("q", H * dim), ("k", H * dim), ("v", H * vdim), ("g", H * vdim)], name="in_proj")
        self.o_proj = Linear(H * vdim, [("o", hidden_size)], name="o")
        self._decay = None

    def sub_parts(self):
        return [("", self.in_proj), ("", self.o_proj)]

    def finalize(self, dtype, device):
        self._decay = (torch.tensor(self.decay, dtype=torch.float32).to(device),
                       torch.tensor([math.log2(d) for d in self.decay], dtype=torch.float64).to(device))

    def cache_needs(self):
        return [StateNeed((self.num_heads, self.dim, self.vdim), "float32", "S")]

    def first_weight(self):
        return self.in_proj.weight

    def forward(self, x, ctx, call):
        H, D, V = self.num_heads, self.dim, self.vdim
        proj = self.in_proj.forward(x, ctx, "retention_proj")
        T = proj.shape[0]
        q, k, v, g = proj.split([H * D, H * D, H * V, H * V], dim=1)
        o = ctx.buffer("head_decay_o", (T, H * V), torch.float32)
        ops.head_decay_scan(q, k, v, ctx.state(call.cache_slot, "S"), ctx.attn_meta, ctx.state_slots, o, H, H, D, V, k_scale=D ** -0.5,
                            decay=self._decay, **_workspaces(ctx, H, D, V))
        gated = ctx.buffer("retention_gated", (T, H * V), ctx.act_dtype)
        ops.gated_group_norm(o, g, None, H, self.norm_eps, gated, gate_first=False)
        return self.o_proj.forward(gated, ctx, "mixer_out")


class Mamba2(Mixer):
    """One projection makes, in this order, a gate z and values x (``heads * vdim`` columns each), keys B and queries C (``groups * state`` each) and
    a step size dt a head.  x, B and C go through one short causal convolution (``taps`` weights and a bias for every channel) and silu.
    Per head, with its group's B and C: g_t = softplus(dt + dt_bias), a_t = exp(-exp(A_log) g_t), k = B, q = C, v = x, and D x joins o.
    silu(z) gates the joined heads in front of an RMS norm over ``norm_groups`` equal parts of the row; then a weight and W_o.  A request's
    slot holds S and the ``taps - 1`` inputs that the convolution still needs.

    Its heads can run inside a mixer that owns the projections (``heads_of``, see ``SideBySide``): ``hosted`` leaves both out."""
    capturable = True

    def __init__(self, hidden_size: int, num_heads: int, vdim: int, state: int, groups: int, taps: int, norm_groups: int, norm_eps: float,
                 hosted: bool = False):
        super().__init__()
        if min(num_heads, vdim, state, groups, taps, norm_groups) < 1 or num_heads % groups or (num_heads * vdim) % norm_groups:
            raise ValueError(f"Mamba2: sizes must be positive, groups divide the heads and norm_groups the inner size: {num_heads} heads of {vdim}, "
                             f"{groups} groups, {norm_groups} norm groups")
        self.hidden_size, self.num_heads, self.vdim, self.state, self.groups, self.taps = hidden_size, num_heads, vdim, state, groups, taps
        self.norm_groups, self.norm_eps = norm_groups, float(norm_eps)
        self.inner = self.heads_width = num_heads * vdim
        self.channels = self.inner + 2 * groups * state                 # what the convolution sees
        self.pieces = [("in", self.inner + self.channels + num_heads)]
        self.in_proj = None if hosted else Linear(hidden_size, self.pieces, name="in_proj")
        self.o_proj = None if hosted else Linear(self.inner, [("o", hidden_size)], name="o")

    def sub_parts(self):
        return [("", part) for part in (self.in_proj, self.o_proj) if part is not None]

    def param_decls(self):
        H, C = self.num_heads, self.channels
        return [ParamDecl("conv", (C, self.taps), init="norm", role="vector"), ParamDecl("conv.b", (C,), role="vector"), ParamDecl("dt_bias", (H,), role="vector"),
                ParamDecl("A_log", (H,), role="vector"), ParamDecl("D", (H,), init="norm", role="vector"),
                ParamDecl("norm", (self.inner,), init="norm", role="vector")]

    def cache_needs(self):
        needs = [StateNeed((self.num_heads, self.state, self.vdim), "float32", "S")]
        if self.taps > 1:
            needs.append(StateNeed((self.taps - 1, self.channels), "float32", "conv"))
        return needs

    def first_weight(self):
        return self.in_proj.weight if self.in_proj is not None else None

    def heads_of(self, proj, ctx, call, out) -> None:
        """``proj`` [T, columns of ``pieces``] float32 -> the joined, gated and normed heads in ``out`` [T, heads_width]."""
        H, P, N, G, inner = self.num_heads, self.vdim, self.state, self.groups, self.inner
        T = proj.shape[0]
        z, u, dt = proj.split([inner, self.channels, H], dim=1)
        xbc = ctx.buffer("mamba_xbc", (T, self.channels), ctx.act_dtype)
        ops.conv_silu(u, self.p("conv"), self.p("conv.b"), ctx.state(call.cache_slot, "conv") if self.taps > 1 else None, ctx.attn_meta,
                      ctx.state_slots, xbc)
        x, B, C = xbc.split([inner, G * N, G * N], dim=1)
        y = ctx.buffer("head_decay_o", (T, inner), torch.float32)
        ops.head_decay_scan(C, B, x, ctx.state(call.cache_slot, "S"), ctx.attn_meta, ctx.state_slots, y, H, G, N, P,
                            dt=(dt, self.p("dt_bias"), self.p("A_log")), skip=self.p("D"), **_workspaces(ctx, H, N, P))
        ops.gated_group_norm(y, z, self.p("norm"), self.norm_groups, self.norm_eps, out, gate_first=True)

    def forward(self, x, ctx, call):
        proj = self.in_proj.forward(x, ctx, "mamba_proj", out_dtype=torch.float32)
        out = ctx.buffer("mamba_heads", (proj.shape[0], self.inner), ctx.act_dtype)
        self.heads_of(proj, ctx, call, out)
        return self.o_proj.forward(out, ctx, "mixer_out")


register_mixer("retention", Retention)
register_mixer("mamba2", Mamba2)
