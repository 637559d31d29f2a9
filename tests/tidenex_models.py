"""Small Tidenex models for the tests: configurations that differ in every size and constant, and random weights.

The writer here knows the tensor names and shapes of the design by itself (it does not ask the engine), draws matrices
as N(0, gain / sqrt(inputs)) so that every layer changes the residual stream noticeably, and lets a test overwrite any
tensor before the folder is written.
"""
from __future__ import annotations

import functools
import json
import os
import tempfile

import torch
from safetensors.torch import save_file


def attn(heads, kv_heads, dim, vdim, diff, rot=None, base=10000.0, scale=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "scale": dim ** -0.5 if scale is None else scale}
    if rot is not None:
        m["rot"] = {"base": base, "dims": rot}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def par(left, right, left_scale, right_scale, temp=None, scale=None, mlp=None):
    """left: (heads, kv heads, dim, vdim); right: (heads, dim, vdim); temp: (coef, every)."""
    lm = dict(zip(("heads", "kv_heads", "dim", "vdim"), left))
    lm["scale"] = left[2] ** -0.5 if scale is None else scale
    if temp is not None:
        lm["q_temp"] = dict(zip(("coef", "every"), temp))
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": lm, "right": dict(zip(("heads", "dim", "vdim"), right)),
                                                      "left_scale": left_scale, "right_scale": right_scale}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(vocab, width, layers, eps=1e-5, loop=None):
    c = {"architecture": "Tidenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# A: the loop sits in the middle, holds both kinds of layer and a layer without feed-forward; values wider than keys, one parallel
#    layer first and one last
A = config(101, 64, [
    par((4, 2, 16, 24), (2, 16, 24), 0.7, 1.3, temp=(0.25, 20), mlp=dense(96)),
    attn(4, 2, 16, 40, 0.45, rot=8, base=500.0, mlp=dense(80)),
    par((6, 3, 24, 8), (4, 8, 40), 1.5, -0.5, temp=(0.6, 7), mlp=None),
    attn(2, 1, 24, 16, 0.2, rot=24, base=90.0, mlp=dense(72)),
    par((2, 2, 8, 16), (1, 24, 8), 0.9, 0.4, mlp=dense(40)),
], eps=1e-6, loop=(1, 3, 3))
# B: no size a multiple of 8; no rotation in one layer; the loop covers the first layers; equal query and kv heads
B = config(75, 52, [
    attn(3, 3, 10, 9, 0.8, rot=6, base=300.0, mlp=dense(70)),
    par((3, 1, 7, 5), (3, 10, 7), 1.0, 1.0, temp=(1.5, 33), scale=0.5, mlp=dense(22)),
    attn(6, 2, 5, 14, -0.3, mlp=None),
], eps=2e-5, loop=(0, 2, 2))
# C: the sizes of tensor-core kernels without any filling (maps of 64 under values of 128; heads of 64 and of 128), no loop
C = config(130, 128, [
    attn(8, 2, 64, 128, 0.35, rot=64, base=1e6, mlp=dense(256)),
    par((8, 2, 64, 64), (2, 64, 64), 0.8, 1.2, temp=(0.1, 40), mlp=dense(192)),
    par((4, 1, 128, 128), (2, 64, 128), 0.5, 0.9, temp=(0.4, 64), mlp=None),
    attn(4, 4, 32, 64, 0.65, rot=16, base=1e4, mlp=dense(128)),
])
# D: rows that tensor-core kernels take only when filled up (maps of 40 and 16, heads of 72 and 32), one head everywhere in the
#    last layer, heads too wide for them in the third, one looped layer, pages of 32
D = config(64, 80, [
    attn(4, 2, 40, 72, 0.5, rot=20, base=2000.0, mlp=dense(104)),
    par((8, 2, 72, 32), (2, 32, 56), 1.2, 0.8, temp=(0.3, 50), mlp=dense(88)),
    attn(2, 2, 80, 96, 0.15, rot=32, base=700.0, mlp=None),
    attn(1, 1, 16, 32, 0.7, rot=2, base=50.0, mlp=dense(24)),
    par((1, 1, 32, 48), (1, 8, 16), 0.6, 1.1, temp=(0.2, 1), mlp=dense(56)),
], loop=(1, 2, 4))

ALL = {"A": (A, 1, 16), "B": (B, 2, 8), "C": (C, 3, 16), "D": (D, 4, 32)}        # config, seed, page size


def tensors(cfg: dict, seed: int, gain: float = 1.2) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(rows, cols, k=gain):
        return torch.randn(rows, cols, generator=g) * (k / cols ** 0.5)

    def around(n, mean, std):
        return mean + std * torch.randn(n, generator=g)
    t = {"embed": torch.randn(cfg["vocab"], W, generator=g) * 0.8, "final.norm": around(W, 1.0, 0.3), "final.norm.b": around(W, 0.0, 0.2)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm2"):
            t[p + n], t[p + n + ".b"] = around(W, 1.0, 0.3), around(W, 0.0, 0.3)
        if layer["type"] == "attention":
            H, G, Dk, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            t[p + "mix.q"], t[p + "mix.k"], t[p + "mix.v"] = mat(2 * H * Dk, W, 1.5), mat(2 * G * Dk, W, 1.5), mat(G * Dv, W, 1.5)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                t[p + "mix." + n] = around(Dk, 0.0, 0.3)
            t[p + "mix.o"] = mat(W, H * Dv, 1.2)
        else:
            a = m["left"]
            H, G, Dk, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "mix.left."
            for n, rows in (("q", H * Dk), ("k", G * Dk), ("v", G * Dv)):
                t[q + n], t[q + n + ".b"] = mat(rows, W, 1.5), around(rows, 0.0, 0.4)
            t[q + "q.norm"], t[q + "k.norm"] = around(H * Dk, 1.0, 0.4), around(G * Dk, 1.0, 0.4)
            t[q + "r1"], t[q + "r2"] = torch.rand(H, generator=g) * 1.5 + 0.05, torch.rand(H, generator=g) * 0.5 + 0.02
            t[q + "o"], t[q + "o.b"] = mat(W, H * Dv, 1.2), around(W, 0.0, 0.3)
            b = m["right"]
            H, Dk, Dv = b["heads"], b["dim"], b["vdim"]
            q = p + "mix.right."
            t[q + "q"], t[q + "f"], t[q + "v"] = mat(H * Dk, W, 1.5), mat(H * Dk, W, 2.0), mat(H * Dv, W, 1.5)
            t[q + "f.b"] = around(H * Dk, 2.0, 2.0)
            t[q + "lower"] = torch.rand(H * Dk, generator=g) * 0.9 * (torch.rand(H * Dk, generator=g) > 0.25)
            t[q + "norm"] = around(Dv, 1.0, 0.3)
            t[q + "o"] = mat(W, H * Dv, 1.2)
        if layer["mlp"] is None:
            del t[p + "norm2"], t[p + "norm2.b"]
        else:
            t[p + "mlp.up"], t[p + "mlp.down"] = mat(layer["mlp"]["ff"], W, 1.6), mat(W, layer["mlp"]["ff"], 1.4)
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def write_folder(cfg: dict, weights: dict[str, torch.Tensor]) -> str:
    d = tempfile.mkdtemp(prefix="me_tidenex_")
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(d, "model.safetensors"))
    return d


@functools.lru_cache(maxsize=None)
def folder(name: str) -> str:
    cfg, seed, _ = ALL[name]
    return write_folder(cfg, tensors(cfg, seed))
