"""Each mechanism of Tidenex alone: the kernels behind it against the plain function, on inputs made so that a fault shows."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_tidenex as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
ATOL = {"float32": 2e-5, "bfloat16": 2e-2}
RTOL = {"float32": 1e-5, "bfloat16": 1e-2}


def _ops():
    from mini_engine_b200 import ops
    ops.require_extension()
    return ops


def g(seed):
    return torch.Generator().manual_seed(seed)


def _meta(lens, contexts):
    """Step metadata as the kernels read it: requests that bring one token come first."""
    D = sum(1 for n in lens if n == 1)
    assert all(n == 1 for n in lens[:D]) and all(n > 1 for n in lens[D:])
    cu = np.concatenate(([0], np.cumsum(lens))).astype(np.int32)
    lists = {}
    for tq in _ops().ATTN_TILE_SIZES:
        tiles = [(b, q0) for b in range(D, len(lens)) for q0 in range(0, lens[b], tq)]
        lists[tq] = (torch.tensor(tiles or [(0, 0)], dtype=torch.int32, device=DEV), len(tiles))
    return SimpleNamespace(cu_seqlens=torch.tensor(cu, device=DEV), context_lens=torch.tensor(contexts, dtype=torch.int32, device=DEV),
                           num_reqs=len(lens), num_tokens=int(sum(lens)), num_decodes=D, tile_lists=lists,
                           max_context_len=max(contexts), num_tiles=sum(n for _, n in lists.values()),
                           workspace=lambda name, shape, dtype: torch.empty(shape, dtype=dtype, device=DEV),
                           error_flag=torch.zeros(4, dtype=torch.int32, device=DEV), scratch_context_len=0,
                           typical_context_len=max(contexts))


# ---- the recurrence -----------------------------------------------------------------------------------
class _Hgrn:
    """The launches of the recurrence and its norm over steps of several requests with state slots."""

    def __init__(self, H, D, V, seed, W=32, slots=3, bias_mean=1.0, bias_std=3.0, eps=1e-5):
        r = lambda rows, k, s: torch.randn(rows, W, generator=g(seed + s)) * (k / W ** 0.5)
        self.m = {"heads": H, "dim": D, "vdim": V}
        self.w = {"q": r(H * D, 2.0, 1), "f": r(H * D, 2.0, 2), "v": r(H * V, 1.5, 3), "o": torch.eye(H * V),
                  "f.b": bias_mean + bias_std * torch.randn(H * D, generator=g(seed + 4)),
                  "lower": torch.rand(H * D, generator=g(seed + 5)) * (torch.rand(H * D, generator=g(seed + 6)) > 0.4),
                  "norm": torch.rand(V, generator=g(seed + 7)) + 0.5}
        self.eps = eps
        self.S = torch.full((slots, H, D, V), float("nan"), device=DEV)

    def plain(self, h):
        return plain.hgrn2(h.double(), {"x." + k: v.double() for k, v in self.w.items()}, "x.", self.m, self.eps)[0]

    def project(self, h):
        return h.to(DEV) @ torch.cat([self.w[k] for k in ("q", "f", "v")]).to(DEV).T

    def step(self, proj, lens, contexts, slots):
        """The projections lie in the middle of wider rows, the results among columns of someone else."""
        ops = _ops()
        H, D, V = self.m["heads"], self.m["dim"], self.m["vdim"]
        T, C = proj.shape
        wide = torch.full((T, C + 11), float("nan"), device=DEV)
        wide[:, 3:3 + C] = proj
        meta = _meta(list(lens), list(contexts))
        runs = ops.gla_chunk_count(meta)
        o = torch.full((T, H * V), float("nan"), device=DEV)
        ops.gla_scan(wide[:, 3:3 + C], {"q": 0, "k": H * D, "v": 2 * H * D}, torch.full((T, H * D), float("nan"), device=DEV), self.S, meta,
                     torch.tensor(slots, dtype=torch.int32, device=DEV), o, H, D, V, 1.0,
                     scores=torch.full((T, H, ops.GLA_CHUNK), float("nan"), device=DEV) if runs else None,
                     chunk_states=torch.full((max(runs, 1), H, D, V), float("nan"), device=DEV) if runs else None,
                     gate=(self.w["f.b"].to(DEV), self.w["lower"].to(DEV)))
        out = torch.full((T, H * V + 6), 7.0, device=DEV)
        ops.mlstm_out(o, wide, 0, self.w["norm"].to(DEV), self.eps, out[:, 4:4 + H * V], H, V, shared_weight=True, gate=None)
        assert (out[:, :4] == 7.0).all() and (out[:, 4 + H * V:] == 7.0).all()
        return out[:, 4:4 + H * V].cpu()

    def sequence(self, h, cuts, slot):
        outs, pos, proj = [], 0, self.project(h)
        for c in cuts:
            outs.append(self.step(proj[pos:pos + c], [c], [pos + c], [slot]))
            pos += c
        return torch.cat(outs)


@pytest.mark.parametrize("H, D, V", [(2, 16, 32), (3, 24, 40), (1, 72, 8), (2, 7, 5), (2, 64, 128), (1, 130, 70)])
def test_recurrence_against_the_plain_one_and_cut_anywhere(H, D, V):
    run = _Hgrn(H, D, V, seed=H * 100 + D)
    h = torch.randn(200, 32, generator=g(H + D + V))
    ref = run.plain(h)
    whole = run.sequence(h, [200], 1)                                    # three runs of 64 tokens and a rest of 8
    single = run.sequence(h, [1] * 200, 2)
    cut = run.sequence(h, [2, 1, 30, 2, 64, 1, 65, 35], 0)
    for got in (whole, single, cut):
        assert torch.allclose(got.double(), ref, atol=1e-4, rtol=3e-4)
    assert torch.allclose(whole, single, atol=5e-5, rtol=1e-4) and torch.allclose(whole, cut, atol=5e-5, rtol=1e-4)
    ops = _ops()
    ops.gla_chunks = False
    try:                                                                 # token by token, a token's arithmetic is the same wherever
        assert torch.equal(run.sequence(h, [200], 1), single)            # the sequence was cut
    finally:
        ops.gla_chunks = True


def test_recurrence_of_unequal_requests_with_slots_used_again():
    run = _Hgrn(3, 24, 40, seed=77, slots=5)
    totals, first = [90, 31, 140, 131, 66], [89, 30, 70, 1, 64]
    hs = [torch.randn(n, 32, generator=g(200 + i)) for i, n in enumerate(totals)]
    refs, projs, slots = [run.plain(h) for h in hs], [run.project(h) for h in hs], [4, 0, 2, 3, 1]

    def check(order, lo, hi):
        lens = [hi[i] - lo[i] for i in order]
        out = run.step(torch.cat([projs[i][lo[i]:hi[i]] for i in order]), lens, [hi[i] for i in order], [slots[i] for i in order])
        at = 0
        for i, n in zip(order, lens):
            assert torch.allclose(out[at:at + n].double(), refs[i][lo[i]:hi[i]], atol=1e-4, rtol=3e-4)
            at += n
    check([3, 0, 1, 2, 4], [0] * 5, first)
    check([0, 1, 4, 2, 3], first, totals)
    out = run.step(torch.cat([projs[2][:100], projs[0][:65]]), [100, 65], [100, 65], [4, 2])      # what the slots held must not show
    assert torch.allclose(out[:100].double(), refs[2][:100], atol=1e-4, rtol=3e-4)
    assert torch.allclose(out[100:].double(), refs[0][:65], atol=1e-4, rtol=3e-4)


@pytest.mark.parametrize("bias_mean, lower", [(-30.0, 0.0), (-300.0, 0.0), (25.0, 0.0), (60.0, 0.0), (0.0, 0.999), (-8.0, 0.0)])
def test_recurrence_gates_that_forget_at_once_or_never(bias_mean, lower):
    """Gates of 0 in float32 (a channel holds the last value alone), gates so close to 1 that almost nothing is written, and a
    lower bound that leaves a thousandth: no overflow, no NaN, and the plain result."""
    run = _Hgrn(2, 16, 24, seed=5, bias_mean=bias_mean, bias_std=2.0, eps=1e-12)
    run.w["lower"][:] = lower
    h = torch.randn(150, 32, generator=g(9))
    ref = run.plain(h)
    for cuts, slot in (([150], 0), ([1] * 150, 1), ([70, 2, 78], 2)):
        got = run.sequence(h, cuts, slot)
        assert torch.isfinite(got).all()
        assert torch.allclose(got.double(), ref, atol=5e-4, rtol=2e-3)


def test_recurrence_a_slow_channel_carries_the_first_token_across_many_runs():
    """One channel is written by the first token alone (its gate is 1/2 there and 1 - 1e-7 or so after it) and read by the last token
    alone: the result is the first token's value, carried by the state's walk over six runs of 64 tokens."""
    run = _Hgrn(1, 8, 16, seed=21, eps=1e-12)
    w, T = run.w, 401
    w["q"][:], w["f"][3], w["lower"][:] = 0, 0, 0
    w["f.b"][3] = 30.0                                   # channel 3 keeps everything ...
    h = torch.randn(T, 32, generator=g(22))
    h[:, 0] = 0
    h[0, 0] = 1.0
    h[T - 1, 1] = 4.0
    h[:T - 1, 1] = 0
    w["f"][3, 0] = -30.0                                 # ... but at the first token
    w["q"][3, 1] = 3.0                                   # read by the last one alone
    ref = run.plain(h)
    v0 = (w["v"].double() @ h[0].double())
    assert torch.allclose(ref[T - 1], v0 / v0.square().mean().sqrt() * w["norm"].double(), atol=1e-6)
    for cuts in ([T], [300, 101], [400, 1], [1] * T):
        assert torch.allclose(run.sequence(h, cuts, 0)[T - 1].double(), ref[T - 1], atol=1e-4, rtol=1e-4)


# ---- attention -----------------------------------------------------------------------------------------
def _paged(keys, values, ps, row, dtype, seed):
    """The keys and values of several requests in pages handed out in a shuffled order, NaN where nothing was written, zeros
    behind a key or value: [pages, 2, kv heads, page, row]."""
    need = [(k.shape[0] + ps - 1) // ps for k in keys]
    pages = sum(need) + 3
    G, D, V = keys[0].shape[1], keys[0].shape[2], values[0].shape[2]
    pool = torch.full((pages, 2, G, ps, row), float("nan"), dtype=dtype, device=DEV)
    perm = torch.randperm(pages, generator=g(seed)).tolist()
    bt = torch.full((len(keys), max(need)), -1, dtype=torch.int32)
    for b, (k, v) in enumerate(zip(keys, values)):
        for i in range(need[b]):
            page = bt[b, i] = perm.pop()
            n = k[i * ps:(i + 1) * ps].shape[0]
            pool[page, :, :, :n] = 0
            pool[page, 0, :, :n, :D] = k[i * ps:(i + 1) * ps].transpose(0, 1).to(dtype).to(DEV)
            pool[page, 1, :, :n, :V] = v[i * ps:(i + 1) * ps].transpose(0, 1).to(dtype).to(DEV)
    return pool, bt.to(DEV)


def _case(dtype, H, G, D, V, ps, lens, contexts, seed, biased=False, pairs=None, boost=None, scale=0.37, window=None):
    """Runs the attention on requests whose last ``lens`` tokens are this step's queries; (got, reference) per request.  ``pairs``
    = (lambda, gain, eps): every head has two maps of D elements."""
    ops, dt, M = _ops(), DT[dtype], 2 if pairs else 1
    qs = [torch.randn(c, H, M * D, generator=g(seed + i)) for i, c in enumerate(contexts)]
    ks = [torch.randn(c, G, M * D, generator=g(seed + 10 + i)) for i, c in enumerate(contexts)]
    vs = [torch.randn(c, G, V, generator=g(seed + 20 + i)) for i, c in enumerate(contexts)]
    r1, r2 = torch.rand(H, generator=g(seed + 30)) * 2, torch.rand(H, generator=g(seed + 31)) * 0.5 + 0.01
    if boost:
        boost(qs, ks)
    qs, ks, vs = ([t.to(dt).float() for t in ts] for ts in (qs, ks, vs))       # what the kernel is given, exactly
    row = ops.padded_head(max(M * D, V))
    pool, bt = _paged(ks, vs, ps, row, dt, seed)
    meta = _meta(list(lens), list(contexts))
    q = torch.zeros(sum(lens), H * M, row)
    for m in range(M):
        q[:, m::M, m * D:(m + 1) * D] = torch.cat([qq[c - n:, :, m * D:(m + 1) * D] for qq, n, c in zip(qs, lens, contexts)])
    wide = torch.full((sum(lens), H * V + 24), 7.0, dtype=dt, device=DEV)      # the results go to columns of a wider tensor
    out = wide[:, 8:8 + H * V]
    ops.sink_attention(q.view(sum(lens), -1).to(dt).to(DEV), None, out, pool, ps, bt, meta, H * M, G, row, V, scale, window, False, padded=True,
                       bias=(r1.to(DEV), r2.to(DEV)) if biased else None, pairs=pairs)
    assert not meta.error_flag.any() and (wide[:, :8] == 7.0).all() and (wide[:, 8 + H * V:] == 7.0).all()
    res, at = [], 0
    for qq, kk, vv, n, c in zip(qs, ks, vs, lens, contexts):
        qd, kd, vd = qq.double(), kk.double(), vv.double()
        bias = (lambda h, d: r1[h].double() * torch.log(1 + r2[h].double() * d)) if biased else None
        if window is not None:
            far = lambda h, d: torch.where(d >= window, torch.inf, 0.0)
            bias = (lambda b: (lambda h, d: (b(h, d) if b else 0) + far(h, d)))(bias)
        if pairs:
            a1, a2 = (plain.causal_attention(qd[..., i * D:(i + 1) * D], kd[..., i * D:(i + 1) * D], vd, scale, bias) for i in (0, 1))
            ref = plain.differential_combine(a1, a2, pairs[0], 1 - pairs[1], pairs[2])
        else:
            ref = plain.causal_attention(qd, kd, vd, scale, bias)
        res.append((out[at:at + n].float().cpu().double(), ref[c - n:].reshape(n, H * V)))
        at += n
    return res


SHAPES = [(4, 2, 16, 24, 16), (3, 1, 10, 9, 8), (8, 2, 64, 64, 16), (6, 2, 40, 56, 64), (4, 4, 128, 128, 32), (2, 2, 80, 104, 16), (16, 1, 32, 96, 128),
          (2, 1, 144, 40, 16)]
LENS, CONTEXTS = (1, 1, 1, 70, 45, 2, 150), (1, 97, 300, 70, 211, 130, 150)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, D, V, ps", SHAPES)
def test_attention_with_a_distance_bias(dtype, H, G, D, V, ps):
    """Single tokens (first in the batch), a prompt from position 0, portions that start in the middle of a page, a portion of two."""
    for got, ref in _case(dtype, H, G, D, V, ps, LENS, CONTEXTS, seed=H * D, biased=True):
        assert torch.allclose(got, ref, atol=ATOL[dtype], rtol=RTOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_attention_with_a_distance_bias_and_a_window(dtype):
    for got, ref in _case(dtype, 4, 2, 64, 64, 16, LENS, CONTEXTS, seed=3, biased=True, window=50):
        assert torch.allclose(got, ref, atol=ATOL[dtype], rtol=RTOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("lam", [0.55, -0.4])
@pytest.mark.parametrize("H, G, D, V, ps", [(4, 2, 8, 24, 16), (3, 1, 5, 9, 8), (8, 2, 64, 128, 16), (6, 2, 20, 40, 64), (4, 4, 32, 64, 32),
                                            (2, 2, 40, 104, 16), (12, 1, 16, 64, 128), (2, 1, 72, 40, 16)])
def test_differential_attention(dtype, H, G, D, V, ps, lam):
    # (the difference of two close results is normed, which magnifies what bfloat16 rounds in each of them)
    tol = dict(atol=5e-5, rtol=1e-4) if dtype == "float32" else dict(atol=6e-2, rtol=2e-2)
    for got, ref in _case(dtype, H, G, D, V, ps, LENS, CONTEXTS, seed=H * D + 1, pairs=(lam, 0.7, 1e-5)):
        assert torch.allclose(got, ref, **tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("biased", [True, False])
@pytest.mark.parametrize("D, ps, j_of", [(16, 16, lambda p: 0), (64, 16, lambda p: 127), (64, 64, lambda p: 128), (40, 8, lambda p: p - 1),
                                         (64, 16, lambda p: p), (128, 32, lambda p: 15), (64, 16, lambda p: 16), (64, 128, lambda p: p // 128 * 128)])
def test_one_sharp_key(dtype, biased, D, ps, j_of):
    """One key gets a score far above the others: the first one, at a page's or a tile's edge, the newest, the one before it.  With pairs
    only the second map has it, which a mixed-up map would show."""
    def boost(qs, ks):
        for r, (qq, kk) in enumerate(zip(qs, ks)):
            p = qq.shape[0] - 1 - 50 * r                        # the decoded token; a token inside the other request's portion
            a = 0 if biased else D
            kk[j_of(p), :, a:a + D] = qq[p, 0:1, a:a + D] * (40.0 / 0.37) / (qq[p, 0, a:a + D] ** 2).sum()
    kw = dict(biased=True) if biased else dict(pairs=(0.8, 1.0, 1e-5))
    for got, ref in _case(dtype, 2, 1, D, D if biased else 64, ps, (1, 60), (331, 331), seed=11 + D, boost=boost, **kw):
        assert torch.allclose(got, ref, atol=ATOL[dtype] * (1 if biased else 3), rtol=RTOL[dtype] * 2)


def test_bias_at_long_distances():
    """Thousands of keys, a few partitions and tiles of 128 keys: the bias of a far key is that of its own distance."""
    for dtype in ("float32", "bfloat16"):
        for got, ref in _case(dtype, 2, 1, 64, 64, 16, (1, 40), (2900, 2100), seed=5, biased=True):
            assert torch.allclose(got, ref, atol=ATOL[dtype] / 2, rtol=RTOL[dtype])


# ---- between the projection and the attention -----------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, D, V", [(4, 2, 16, 24), (3, 1, 10, 9), (2, 2, 64, 64), (5, 5, 40, 72), (1, 1, 200, 8),
                                         (32, 8, 128, 128), (6, 2, 100, 132), (20, 10, 36, 8), (48, 48, 4, 8)])
@pytest.mark.parametrize("extra", [5, 8])
def test_norm_over_the_whole_projection_temperature_and_scaled_values(dtype, H, G, D, V, extra):
    """Heads of very different size (a norm by head would make them equal), rows that can be read four values at a time and rows that cannot, positions at and around the temperature's steps, rows
    filled with zeros up to their width."""
    ops, dt, T, ps, eps = _ops(), DT[dtype], 41, 8, 1e-5
    C = H * D + G * (D + V)
    proj = torch.randn(T, C + extra, generator=g(1)) * 2                       # columns beyond q|k|v belong to someone else
    for h in range(H):
        proj[:, h * D:(h + 1) * D] *= 3.0 ** -h
    b = torch.randn(C, generator=g(2))
    qw, kw = torch.rand(H * D, generator=g(3)) + 0.2, torch.rand(G * D, generator=g(4)) + 0.2
    positions = torch.tensor([0, 5, 6, 7, 12, 13, 14, 70001, 1 << 20] + list(range(500, 500 + T - 9)), dtype=torch.int32)
    x = proj[:, :C].double() + b.double()
    q = plain.over_rms(x[:, :H * D], eps) * qw.double() * plain.temperature(positions.double(), 0.4, 7)[:, None]
    k = plain.over_rms(x[:, H * D:(H + G) * D], eps) * kw.double()
    row = ops.padded_head(max(D, V))
    pool = torch.full((8, 2, G, ps, row), float("nan"), dtype=dt, device=DEV)
    slots = torch.randperm(8 * ps, generator=g(5))[:T].to(torch.int32)
    q_out = torch.full((T, H * row), float("nan"), dtype=dt, device=DEV)
    ops.attn_prep(proj.to(DEV), b.to(DEV), qw.to(DEV), kw.to(DEV), "row", eps, None, positions.to(DEV), slots.to(DEV), q_out, pool, ps, H, G, D, V,
                  temperature=(0.4, 7.0), v_scale=-0.6)
    tol = dict(atol=2e-5, rtol=1e-5) if dtype == "float32" else dict(atol=2e-2, rtol=1e-2)
    got = q_out.float().cpu().double().view(T, H, row)
    assert torch.allclose(got[..., :D], q.view(T, H, D), **tol) and (got[..., D:] == 0).all()
    rows = pool.float().cpu().double()
    for t in range(T):
        page, off = int(slots[t]) // ps, int(slots[t]) % ps
        assert torch.allclose(rows[page, 0, :, off, :D], k[t].view(G, D), **tol) and (rows[page, 0, :, off, D:] == 0).all()
        assert torch.allclose(rows[page, 1, :, off, :V], -0.6 * x[t, (H + G) * D:].view(G, V), **tol) and (rows[page, 1, :, off, V:] == 0).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, D, V, rot", [(4, 2, 8, 24, 6), (3, 3, 10, 9, 10), (4, 1, 64, 128, 32), (2, 1, 24, 20, 0), (1, 1, 80, 96, 2),
                                             (32, 8, 64, 128, 64), (5, 5, 20, 100, 16), (2, 2, 12, 256, 8), (40, 8, 120, 40, 120)])
@pytest.mark.parametrize("T", [37, 139])
def test_two_maps_a_head_are_rotated_each_by_itself(dtype, H, G, D, V, rot, T):
    """Short and long steps run different kernels (a warp a map, a block a token)."""
    ops, dt, ps = _ops(), DT[dtype], 8
    C = 2 * H * D + G * (2 * D + V)
    proj = torch.randn(T, C, generator=g(1)) * 2
    positions = torch.tensor([0, 1, 2, 3, 70001, 1 << 20] + list(range(500, 500 + T - 6)), dtype=torch.int32)
    q, k = proj[:, :2 * H * D].double().view(T, H, 2, D), proj[:, 2 * H * D:2 * (H + G) * D].double().view(T, G, 2, D)
    q, k = plain.rotate(q, positions, rot, 3000.0), plain.rotate(k, positions, rot, 3000.0)
    freq = torch.tensor([3000.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device=DEV) if rot else None
    row = ops.padded_head(max(2 * D, V))
    pool = torch.full((20, 2, G, ps, row), float("nan"), dtype=dt, device=DEV)
    slots = torch.randperm(20 * ps, generator=g(5))[:T].to(torch.int32)
    slots[7] = -1                                                          # not written
    q_out = torch.full((T, 2 * H * row), float("nan"), dtype=dt, device=DEV)
    ops.attn_prep(proj.to(DEV), None, None, None, None, 1e-5, freq, positions.to(DEV), slots.to(DEV), q_out, pool, ps, H, G, D, V, maps=2)
    tol = dict(atol=2e-5, rtol=1e-5) if dtype == "float32" else dict(atol=2e-2, rtol=1e-2)
    got = q_out.float().cpu().double().view(T, H, 2, row)
    for m in (0, 1):
        assert torch.allclose(got[:, :, m, m * D:(m + 1) * D], q[:, :, m], **tol)
        assert (got[:, :, m, :m * D] == 0).all() and (got[:, :, m, (m + 1) * D:] == 0).all()
    rows = pool.float().cpu().double()
    for t in range(T):
        if t == 7:
            continue
        page, off = int(slots[t]) // ps, int(slots[t]) % ps
        assert torch.allclose(rows[page, 0, :, off, :2 * D], k[t].reshape(G, 2 * D), **tol) and (rows[page, 0, :, off, 2 * D:] == 0).all()
        assert torch.allclose(rows[page, 1, :, off, :V], proj[t, 2 * (H + G) * D:].double().view(G, V), **tol) and (rows[page, 1, :, off, V:] == 0).all()


# ---- the residual sum that takes the embedding along ------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W", [40, 53, 1030, 4100])
def test_residual_sum_with_the_embedding(dtype, W):
    """Tokens by id and by reference to the tokens a step before drew (~j), beside an output and a bias; and the embedding alone."""
    ops, dt, T, V, eps = _ops(), DT[dtype], 9, 17, 1e-6
    x, y, va = torch.randn(T, W, generator=g(W)) + 5.0, torch.randn(T, W, generator=g(W + 1)).to(dt), torch.randn(W, generator=g(W + 2))
    table = torch.randn(V, W, generator=g(W + 3)).to(dt)
    w, b = torch.randn(W, generator=g(W + 4)), torch.randn(W, generator=g(W + 5))
    feedback = torch.tensor([11, 0, 16], dtype=torch.int32)
    ids = torch.tensor([3, 0, 16, ~0, ~2, 5, ~1, 3, 9], dtype=torch.int32)
    real = torch.tensor([3, 0, 16, 11, 16, 5, 0, 3, 9])
    tol = dict(atol=2e-4, rtol=1e-4) if dtype == "float32" else dict(atol=3e-2, rtol=1e-2)
    for outputs, vectors, scale in (([y], [va], 1.0), ([], [], 0.5)):
        want = x.double() + sum(o.double() for o in outputs) + sum(v.double() for v in vectors) + scale * table[real].double()
        res, out = x.to(DEV), torch.empty(T, W, dtype=dt, device=DEV)
        ops.parallel_norm(res, [o.to(DEV) for o in outputs], [v.to(DEV) for v in vectors], eps, (w.to(DEV), b.to(DEV)), out,
                          embedding=(ids.to(DEV), table.to(DEV), feedback.to(DEV), scale))
        assert torch.allclose(res.cpu().double(), want, atol=1e-5)
        assert torch.allclose(out.float().cpu().double(), plain.layer_norm(want, w.double(), b.double(), eps), **tol)


# ---- the feed-forward --------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T, W, F", [(1, 64, 96), (5, 52, 70), (40, 128, 200), (300, 128, 264), (1100, 256, 520), (1500, 512, 6144)])
@pytest.mark.parametrize("in_product", [True, False])
def test_gelu_feed_forward_in_every_kernel_of_its_product(dtype, T, W, F, in_product):
    """One row to many: the products and their activation run different kernels, with the activation as a pass of its own or in the
    product's epilogue."""
    from mini_engine_b200.parts import ActivationMLP
    if dtype == "float32" and T > 500:
        T = 130
    dt = DT[dtype]
    mlp = ActivationMLP(W, F, "gelu", in_product=in_product)
    up, down = (torch.randn(F, W, generator=g(1)) * (2.0 / W ** 0.5)).to(dt), (torch.randn(W, F, generator=g(2)) / F ** 0.5).to(dt)
    mlp.up.params["up"], mlp.down.params["down"] = up.to(DEV), down.to(DEV)
    x = torch.randn(T, W, generator=g(3)).to(dt)
    ctx = SimpleNamespace(act_dtype=dt, error_flag=torch.zeros(4, dtype=torch.int32, device=DEV),
                          buffer=lambda name, shape, dtype, zero=False: torch.zeros(shape, dtype=dtype, device=DEV))
    got = mlp.forward(x.to(DEV), ctx)
    assert not ctx.error_flag.any()
    ref = plain.gelu_mlp(x.double(), {"up": up.double(), "down": down.double()}, "")
    tol = dict(atol=2e-5, rtol=1e-4) if dtype == "float32" else dict(atol=3e-2, rtol=2e-2)
    assert torch.allclose(got.float().cpu().double(), ref, **tol)


def test_gelu_is_the_exact_one():
    """At -3 the exact form and its tanh approximation differ by a tenth."""
    ops = _ops()
    z = torch.linspace(-6, 6, 1000).view(10, 100)
    out = torch.empty(10, 100, device=DEV)
    ops.activation(z.to(DEV), out, "gelu")
    ref = plain.gelu_exact(z.double())
    assert (out.cpu().double() - ref).abs().max() < 1e-6
    approx = 0.5 * z.double() * (1 + torch.tanh((2 / np.pi) ** 0.5 * (z.double() + 0.044715 * z.double() ** 3)))
    assert (approx - ref).abs().max() > 1e-4
