"""Small Kuterax models for the tests: configurations that differ in every size and constant, and random weights.

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


def par(left, right, window, rot, base=10000.0, scaling=(8.0, 256, 16.0, 1.0), scale=None, mlp=None):
    """left: (heads, kv heads, dim, vdim); right: (heads, vdim, state, groups, taps, norm groups); scaling: (factor, original, fast, slow)."""
    lm = dict(zip(("heads", "kv_heads", "dim", "vdim"), left))
    lm["scale"] = left[2] ** -0.5 if scale is None else scale
    lm["rot"] = {"base": base, "dims": rot}
    if scaling is not None:
        lm["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if window is not None:
        lm["mask"] = {"size": window}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": lm, "right": dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), right))}}


def ret(heads, dim, vdim, decay, mlp=None):
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def moe(experts, top, ff, groups=None, scale=1.0, shared=None):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "router": r, "expert": {"ff": ff}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def config(vocab, width, layers, eps=1e-5, loop=None, max_positions=512):
    c = {"architecture": "Kuterax", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# A: the loop sits in the middle and holds both kinds of layer and one without feed-forward; values wider and narrower than keys,
#    part of a head rotated, one group of experts of three kept
A = config(101, 64, [
    ret(2, 16, 24, (0.9, 0.99), mlp=moe(6, 2, 40, groups=(3, 1), scale=1.3, shared=56)),
    par((4, 2, 16, 24), (4, 8, 16, 2, 4, 2), 20, 8, base=500.0, mlp=moe(8, 3, 32, groups=(4, 2), scale=0.7, shared=24)),
    ret(3, 8, 40, (0.5, 0.97, 1.0), mlp=None),
    par((6, 3, 24, 8), (2, 24, 8, 1, 3, 4), 33, 24, scaling=(3.0, 100, 6.0, 0.5), mlp=moe(4, 1, 48, groups=(2, 2), scale=2.0, shared=32)),
], eps=1e-6, loop=(1, 3, 3))
# B: no size a multiple of 8, equal query and kv heads, equal heads and groups, the loop covers the first layers, groups of one expert
B = config(75, 52, [
    par((3, 3, 10, 9), (3, 7, 5, 3, 2, 3), 11, 6, base=90.0, scaling=(1.5, 64, 4.0, 1.0), mlp=moe(5, 2, 22, groups=(5, 3), scale=1.5, shared=30)),
    ret(3, 9, 14, (0.8, 0.95, 0.9), mlp=moe(3, 3, 18, scale=0.6, shared=10)),
    par((3, 1, 7, 5), (2, 5, 11, 1, 5, 1), 16, 2, base=300.0, scale=0.5, mlp=None),
], eps=2e-5, loop=(0, 2, 2))
# C: the sizes of tensor-core kernels without any filling (heads of 64 and of 128), no loop, steps of enough tokens for every
#    kernel of the experts' products
C = config(130, 128, [
    par((8, 2, 64, 64), (4, 64, 64, 2, 4, 2), 100, 64, base=1e6, mlp=moe(8, 4, 64, groups=(2, 1), scale=1.5, shared=128)),
    ret(2, 64, 128, (0.95, 0.998), mlp=moe(4, 2, 128, groups=(2, 2), scale=1.0, shared=64)),
    par((4, 1, 128, 128), (2, 128, 128, 1, 4, 1), 129, 32, base=1e4, scaling=(4.0, 512, 32.0, 1.0), mlp=None),
], max_positions=700)
# D: rows that tensor-core kernels take only when filled up, heads too wide for them in the third layer, a window of one token and
#    one of two pages, conv taps of one and of six, one looped layer, pages of 32, no shared expert in one layer, no YaRN in one
D = config(64, 80, [
    par((4, 2, 40, 72), (4, 16, 24, 4, 1, 8), 7, 20, base=2000.0, mlp=moe(6, 3, 40, groups=(2, 2), scale=1.1, shared=48)),
    par((8, 2, 72, 32), (6, 12, 20, 3, 6, 2), 64, 72, base=50000.0, scaling=(16.0, 128, 8.0, 2.0), mlp=moe(4, 2, 24, groups=(4, 3), scale=1.4, shared=16)),
    par((2, 2, 144, 96), (1, 32, 32, 1, 4, 1), 1, 32, scaling=None, mlp=None),
    ret(1, 72, 8, (0.999,), mlp=moe(2, 1, 56, scale=0.9)),
], loop=(1, 2, 4))

ALL = {"A": (A, 1, 16), "B": (B, 2, 8), "C": (C, 3, 16), "D": (D, 4, 32)}        # config, seed, page size


def tensors(cfg: dict, seed: int, gain: float = 1.2) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(rows, cols, k=gain):
        return torch.randn(rows, cols, generator=g) * (k / cols ** 0.5)

    def around(n, mean, std):
        return mean + std * torch.randn(n, generator=g)
    t = {"embed": torch.randn(cfg["vocab"], W, generator=g) * 0.8, "pos": torch.randn(cfg["max_positions"], W, generator=g) * 0.5,
         "final.norm": around(W, 0.0, 0.3), "head": mat(cfg["vocab"], W, 1.5)}
    if cfg.get("loop"):
        t["loop.in"], t["loop.step"] = mat(W, 2 * W, 1.2), torch.randn(cfg["loop"]["times"], W, generator=g) * 0.5
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        t[p + "norm1"], t[p + "ls1"] = around(W, 0.0, 0.3), around(W, 0.9, 0.3)
        if layer["type"] == "parallel":
            a, q = m["left"], p + "mix.left."
            H, G, Dk, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, rows in (("q", H * Dk), ("k", G * Dk), ("v", G * Dv)):
                t[q + n], t[q + n + ".b"] = mat(rows, W, 1.5), around(rows, 0.0, 0.4)
            t[q + "q.norm"], t[q + "k.norm"] = around(Dk, 1.2, 0.4), around(Dk, 1.2, 0.4)
            t[q + "g"], t[q + "o"] = mat(H, W, 2.0), mat(W, H * Dv, 1.2)
            b, q = m["right"], p + "mix.right."
            H, P, N, Gr = b["heads"], b["vdim"], b["state"], b["groups"]
            inner, C = H * P, H * P + 2 * Gr * N
            t[q + "in"] = mat(inner + C + H, W, 1.5)
            t[q + "conv"], t[q + "conv.b"] = torch.randn(C, b["conv"], generator=g) * 0.6, around(C, 0.1, 0.3)
            t[q + "dt_bias"], t[q + "A_log"], t[q + "D"] = around(H, -2.0, 1.0), around(H, -0.5, 1.0), around(H, 0.7, 0.5)
            t[q + "norm"], t[q + "o"] = around(inner, 1.0, 0.3), mat(W, inner, 1.2)
            t[p + "mix.left.out"], t[p + "mix.right.out"] = around(W, 1.0, 0.3), around(W, 0.8, 0.3)
        else:
            H, Dk, Dv, q = m["heads"], m["dim"], m["vdim"], p + "mix."
            t[q + "q"], t[q + "k"], t[q + "v"] = mat(H * Dk, W, 1.5), mat(H * Dk, W, 1.5), mat(H * Dv, W, 1.5)
            t[q + "g"], t[q + "o"] = mat(H * Dv, W, 1.5), mat(W, H * Dv, 1.2)
        if layer["mlp"] is not None:
            f, q = layer["mlp"], p + "mlp."
            t[p + "ls2"] = around(W, 0.8, 0.3)
            for e in range(f["router"]["experts"]):
                t[f"{q}e{e}.up"], t[f"{q}e{e}.down"] = mat(f["expert"]["ff"], W, 1.6), mat(W, f["expert"]["ff"], 1.2)
            t[q + "router"] = mat(f["router"]["experts"], W, 2.0)
            if f.get("shared"):
                t[q + "shared.up"], t[q + "shared.down"] = mat(f["shared"]["ff"], W, 1.4), mat(W, f["shared"]["ff"], 1.0)
                t[q + "shared.sg"] = mat(1, W, 2.0)
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def write_folder(cfg: dict, weights: dict[str, torch.Tensor]) -> str:
    d = tempfile.mkdtemp(prefix="me_kuterax_")
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(d, "model.safetensors"))
    return d


@functools.lru_cache(maxsize=None)
def folder(name: str) -> str:
    cfg, seed, _ = ALL[name]
    return write_folder(cfg, tensors(cfg, seed))
