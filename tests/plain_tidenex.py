"""A plain, slow Tidenex in float64 torch on the CPU: one function per mechanism, written from the design's equations.

It shares no code with the engine: weights are a dict from disk names to tensors, a sequence is processed whole, the
attention holds the full matrix of scores of a head and the recurrence is a loop over tokens.  Notation: T tokens, W the
model width, H query heads, G key/value heads, D the size of a query or key head (of one map of it in the differential
mixer), Dv of a value head.
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
def layer_norm(x, weight, bias, eps):
    """Over the last axis: distance from the mean, over the root of the mean squared distance (eps inside), then w and b."""
    dev = x - x.mean(-1, keepdim=True)
    return dev / torch.sqrt(dev.square().mean(-1, keepdim=True) + eps) * weight + bias


def over_rms(x, eps):
    """x over the root of its mean square (eps inside), over the last axis."""
    return x / torch.sqrt(x.square().mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu_exact(z):
    """z times the standard normal distribution function at z."""
    return z * 0.5 * torch.erfc(-z / math.sqrt(2.0))


def rotate(x, positions, dims, base):
    """Rotary positions on the first ``dims`` elements of the last axis, element i with element i + dims/2, angle
    position * base^(-2i/dims).  x [T, ..., D]; positions [T]."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = positions.to(x.dtype) * base ** (-2.0 * i / dims)
        shape = (-1,) + (1,) * (x.dim() - 2)
        c, s = torch.cos(a).view(shape), torch.sin(a).view(shape)
        u, v = x[..., i], x[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


# ---- attention ------------------------------------------------------------------------------------
def causal_attention(q, k, v, scale, bias=None):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv].  Query i sees the keys j <= i.  ``bias(h, distance)`` is
    taken off the scaled score of head h at distance i - j."""
    T, H, _ = q.shape
    G = k.shape[1]
    at = torch.arange(T)
    distance = (at[:, None] - at[None, :]).to(q.dtype)
    hidden = distance < 0
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if bias is not None:
            s = s - bias(h, distance.clamp(min=0))
        e = torch.exp(s.masked_fill(hidden, -math.inf) - s.masked_fill(hidden, -math.inf).amax(-1, keepdim=True))
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, g]
    return out


def temperature(positions, coef, every):
    """1 + coef ln(floor((p + 1) / every) + 1)."""
    return 1.0 + coef * torch.log(torch.floor((positions + 1.0) / every) + 1.0)


def biased_attention(h, w, p, m, eps):
    """Biased projections, q and k each normed over their whole row, a temperature on q, a bias by distance, no rotation."""
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = over_rms(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]
    k = over_rms(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]
    v = h @ w[p + "v"].T + w[p + "v.b"]
    if m.get("q_temp"):
        q = q * temperature(torch.arange(T, dtype=h.dtype), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None]
    r1, r2 = w[p + "r1"], w[p + "r2"]
    o = causal_attention(q.view(T, H, D), k.view(T, G, D), v.view(T, G, Dv), m["scale"],
                         lambda hd, d: r1[hd] * torch.log(1.0 + r2[hd] * d))
    return o.reshape(T, H * Dv) @ w[p + "o"].T + w[p + "o.b"]


def differential_lambda(w, p, diff):
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def differential_combine(a1, a2, lam, diff, eps):
    """Per head over its values: a1 - lambda a2, over its root mean square, times (1 - diff)."""
    return over_rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, w, p, m, eps):
    """Two maps a head over the same values; their difference, normed."""
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, 2, D)
    k = (h @ w[p + "k"].T).view(T, G, 2, D)
    v = (h @ w[p + "v"].T).view(T, G, Dv)
    rot = m.get("rot")
    if rot and rot["dims"]:
        at = torch.arange(T)
        q, k = rotate(q, at, rot["dims"], rot["base"]), rotate(k, at, rot["dims"], rot["base"])
    a1, a2 = (causal_attention(q[:, :, i], k[:, :, i], v, m["scale"]) for i in (0, 1))
    o = differential_combine(a1, a2, differential_lambda(w, p, m["diff"]), m["diff"], eps)
    return o.reshape(T, H * Dv) @ w[p + "o"].T


# ---- the recurrence -------------------------------------------------------------------------------
def forget_gate(z, lower):
    """l + (1 - l) sigmoid(z), per channel."""
    return lower + (1.0 - lower) * torch.sigmoid(z)


def gated_recurrence(q, f, v, state=None):
    """q, f [T, H, D], v [T, H, Dv] -> (o [T, H, Dv], last state [H, D, Dv]): S <- f S + (1 - f) v^T, o = S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def hgrn2(h, w, p, m, eps, state=None):
    """A matrix state with the gate as decay and 1 - gate as key; returns (output, last state)."""
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).view(T, H, D)
    f = forget_gate(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"]).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, Dv)
    o, S = gated_recurrence(q, f, v, state)
    return (over_rms(o, eps) * w[p + "norm"]).reshape(T, H * Dv) @ w[p + "o"].T, S


# ---- layers and the model -------------------------------------------------------------------------
def mixer(h, w, p, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "attention":
        return differential_attention(h, w, p, m, eps)
    if layer["type"] == "parallel":
        left = biased_attention(h, w, p + "left.", m["left"], eps)
        right, _ = hgrn2(h, w, p + "right.", m["right"], eps)
        return m["left_scale"] * left + m["right_scale"] * right
    raise ValueError(layer["type"])


def gelu_mlp(h, w, p):
    return gelu_exact(h @ w[p + "up"].T) @ w[p + "down"].T


def layer_runs(cfg):
    """(layer, whether the embedding output joins the stream in front of it) in the order in which layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg, w, tokens, return_layers=False):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer run)."""
    eps = cfg["norm"]["eps"]
    first = w["embed"][torch.as_tensor(tokens)]
    x, after = first, []
    for i, rejoin in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if rejoin:
            x = x + first
        x = x + mixer(layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps), w, p + "mix.", layer, eps)
        if layer.get("mlp"):
            x = x + gelu_mlp(layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps), w, p + "mlp.")
        after.append(x)
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
    return (logits, torch.stack(after)) if return_layers else logits
