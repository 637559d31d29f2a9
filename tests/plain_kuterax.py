"""A plain, slow Kuterax in float64 torch on the CPU: one function per mechanism, written from the design's equations.

It shares no code with the engine: weights are a dict from disk names to tensors, a sequence is processed whole, the
attention holds the full matrix of scores of a head and both recurrences are loops over tokens.  Notation: T tokens, W the
model width, H heads, G key/value heads, D the size of a query or key head, Dv of a value head, N the rows of a
state-space head's state.
"""
from __future__ import annotations

import json
import math
import os

import torch
from safetensors import safe_open


def load_folder(folder: str, dtype=torch.float64):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    w = {}
    with safe_open(os.path.join(folder, "model.safetensors"), "pt", device="cpu") as f:
        for name in f.keys():
            t = f.get_tensor(name)
            w[name] = t.to(dtype) if t.is_floating_point() else t
    return cfg, w


# ---- small pieces ---------------------------------------------------------------------------------
def over_rms(x, eps):
    """x over the root of its mean square (eps inside), over the last axis."""
    return x / torch.sqrt(x.square().mean(-1, keepdim=True) + eps)


def norm_around_zero(x, weight, eps):
    return over_rms(x, eps) * (1.0 + weight)


def over_rms_in_groups(x, groups, eps):
    """Every one of ``groups`` equal parts of the last axis over its own root mean square."""
    return over_rms(x.unflatten(-1, (groups, -1)), eps).flatten(-2)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return z.clamp(min=0) + torch.log1p(torch.exp(-z.abs()))


def yarn_frequencies(dims, base, scaling=None):
    """(frequencies, factor on cosines and sines): plain base^(-2i/dims), or blended with their ``factor``-th part by a ramp over i
    whose ends are where a wavelength fits ``fast`` and ``slow`` times into ``original`` positions."""
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return plain, 1.0

    def index_with_turns(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index_with_turns(scaling["fast"])), 0)
    hi = min(math.ceil(index_with_turns(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_halves(x, positions, freqs, magnitude=1.0):
    """Element i with element i + n of the first 2 n = 2 len(freqs) elements.  x [T, heads, D]; positions [T]."""
    n = len(freqs)
    out = x.clone()
    for i, f in enumerate(freqs):
        a = positions.to(x.dtype) * f
        c, s = (torch.cos(a) * magnitude)[:, None], (torch.sin(a) * magnitude)[:, None]
        u, v = x[..., i], x[..., i + n]
        out[..., i], out[..., i + n] = u * c - v * s, v * c + u * s
    return out


# ---- attention ------------------------------------------------------------------------------------
def window_attention(q, k, v, scale, window, one_more=True):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv].  Query i sees the keys 0 <= i - j < window; ``one_more``: the
    denominator has a one of its own."""
    T, H, _ = q.shape
    G = k.shape[1]
    at = torch.arange(T)
    distance = at[:, None] - at[None, :]
    hidden = (distance < 0) | (distance >= window)
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(hidden, -math.inf)
        top = s.amax(-1, keepdim=True)
        if one_more:
            top = top.clamp(min=0.0)
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True) + (torch.exp(-top) if one_more else 0.0)
        out[:, h] = (e / den) @ v[:, g]
    return out


def attention_branch(h, w, p, m, eps):
    """Biased projections, normed heads, YaRN rotation, a window, a one in the denominator, a gate a head."""
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, Dv)
    q, k = over_rms(q, eps) * w[p + "q.norm"], over_rms(k, eps) * w[p + "k.norm"]
    if m.get("rot"):
        freqs, magnitude = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        at = torch.arange(T)
        q, k = rotate_halves(q, at, freqs, magnitude), rotate_halves(k, at, freqs, magnitude)
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"] if m.get("mask") else T)
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * Dv) @ w[p + "o"].T


# ---- recurrences ----------------------------------------------------------------------------------
def causal_conv(u, taps_weight, bias):
    """out[t] = bias + sum over j of weight[:, j] u[t - taps + 1 + j], zeros before the start.  u [T, C]; weight [C, taps]."""
    T, taps = u.shape[0], taps_weight.shape[1]
    out = bias.expand_as(u).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] = out[back:] + u[:T - back] * taps_weight[:, j]
    return out


def state_space_scan(x, B, C, dt, A_log, D, state=None):
    """x [T, H, P], B, C [T, G, N], dt [T, H] -> (y [T, H, P], last state [H, N, P])."""
    T, H, P = x.shape
    G, N = B.shape[1], B.shape[2]
    S = torch.zeros(H, N, P, dtype=x.dtype) if state is None else state.clone()
    y = torch.empty_like(x)
    of_head = torch.arange(H) // (H // G)
    rate = torch.exp(A_log)
    for t in range(T):
        keep = torch.exp(-rate * dt[t])
        S = keep[:, None, None] * S + (dt[t][:, None] * B[t][of_head])[:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t][of_head][:, :, None]).sum(1) + D[:, None] * x[t]
    return y, S


def state_space_branch(h, w, p, m, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xBC, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = silu(causal_conv(xBC, w[p + "conv"], w[p + "conv.b"])).split([inner, G * N, G * N], dim=-1)
    y, _ = state_space_scan(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    y = over_rms_in_groups(y.reshape(T, inner) * silu(z), m["norm_groups"], eps) * w[p + "norm"]
    return y @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    left = attention_branch(h, w, p + "left.", m["left"], eps)
    right = state_space_branch(h, w, p + "right.", m["right"], eps)
    return 0.5 * (over_rms(left, eps) * w[p + "left.out"] + over_rms(right, eps) * w[p + "right.out"])


def retention_scan(q, k, v, decay, state=None):
    """q, k [T, H, D], v [T, H, Dv], decay [H] -> (o [T, H, Dv], last state [H, D, Dv])."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    a = torch.as_tensor(decay, dtype=q.dtype)
    for t in range(T):
        S = a[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def retention_mixer(h, w, p, m, eps):
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (h @ w[p + "q"].T).view(T, H, D), (h @ w[p + "k"].T).view(T, H, D) * D ** -0.5
    v = (h @ w[p + "v"].T).view(T, H, Dv)
    o, _ = retention_scan(q, k, v, m["decay"])
    return (over_rms(o, eps).reshape(T, H * Dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward ---------------------------------------------------------------------------------
def squared_relu_mlp(h, w, p):
    return (h @ w[p + "up"].T).clamp(min=0).square() @ w[p + "down"].T


def route(z, top, groups, keep, scale):
    """One token's logits [E] -> (chosen experts, their weights): softmax over all, the best ``keep`` of ``groups`` groups by their
    largest score, the ``top`` largest scores among those, times ``scale``."""
    E = z.shape[0]
    n = E // groups
    s = torch.softmax(z, -1)
    of_group = s.view(groups, n).amax(-1)
    kept = sorted(range(groups), key=lambda g: (-of_group[g].item(), g))[:keep]
    allowed = [e for e in range(E) if e // n in kept]
    chosen = sorted(allowed, key=lambda e: (-s[e].item(), e))[:top]
    return chosen, [s[e] * scale for e in chosen]


def routed_experts(h, w, p, mlp, chosen_out=None):
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ w[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, weights = route(z[t], r["top"], g["count"], g["keep"], r["scale"])
        if chosen_out is not None:
            chosen_out.append(chosen)
        for e, s in zip(chosen, weights):
            out[t] = out[t] + s * squared_relu_mlp(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * squared_relu_mlp(h, w, p + "shared.")
    return out


# ---- layers and the model -------------------------------------------------------------------------
def mixer(h, w, p, layer, eps):
    if layer["type"] == "parallel":
        return parallel_mixer(h, w, p, layer["mixer"], eps)
    if layer["type"] == "retention":
        return retention_mixer(h, w, p, layer["mixer"], eps)
    raise ValueError(layer["type"])


def layer_runs(cfg):
    """(layer, number of the pass that starts in front of it or None) in the order in which layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def join_pass(x, first, w, t):
    """What stands in front of pass t: W_in [x; embedding output] plus the pass's vector."""
    return torch.cat([x, first], -1) @ w["loop.in"].T + w["loop.step"][t]


def forward(cfg, w, tokens, return_layers=False):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer run)."""
    eps = cfg["norm"]["eps"]
    first = w["embed"][torch.as_tensor(tokens)] + w["pos"][:len(tokens)]
    x, after = first, []
    for i, t in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = join_pass(x, first, w, t)
        h = norm_around_zero(x, w[p + "norm1"], eps)
        y = mixer(h, w, p + "mix.", layer, eps) * w[p + "ls1"]
        if layer.get("mlp"):
            y = y + routed_experts(h, w, p + "mlp.", layer["mlp"]) * w[p + "ls2"]
        x = x + y
        after.append(x)
    logits = norm_around_zero(x, w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(after)) if return_layers else logits
