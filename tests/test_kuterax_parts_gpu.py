"""Each mechanism of Kuterax alone: the kernels behind it against the plain function, on inputs made so that a fault shows."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_kuterax as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
both = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


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


# ---- the recurrences ------------------------------------------------------------------------------------
class _Scan:
    """The recurrence's launches over steps of several requests with state slots.  ``constant``: a decay a head; else dt, A_log and D."""

    def __init__(self, H, G, D, V, dtype, constant, seed=0, slots=3, decay=None, a_log=None, dt_bias=None):
        self.H, self.G, self.D, self.V, self.dt, self.constant = H, G, D, V, DT[dtype], constant
        self.decay = torch.rand(H, generator=g(seed)) * 0.5 + 0.5 if decay is None else torch.tensor(decay)
        self.a_log = torch.randn(H, generator=g(seed + 1)) if a_log is None else torch.full((H,), float(a_log))
        self.dt_bias = torch.randn(H, generator=g(seed + 2)) - 1.0 if dt_bias is None else torch.full((H,), float(dt_bias))
        self.skip = torch.randn(H, generator=g(seed + 3))
        self.S = torch.full((slots, H, D, V), float("nan"), device=DEV)
        self.pad = 4                                                     # columns in front of and between q, k and v

    def inputs(self, T, seed):
        q, k = (torch.randn(T, self.G * self.D, generator=g(seed + i)) / self.D ** 0.25 for i in (0, 1))
        v, dt = torch.randn(T, self.H * self.V, generator=g(seed + 2)), torch.randn(T, self.H, generator=g(seed + 3)) * 1.5
        return [t.to(self.dt).float() for t in (q, k, v)] + [dt]           # what the kernels are given, exactly

    def plain(self, x):
        q, k, v, dt = (t.double() for t in x)
        T, H, G, D, V = q.shape[0], self.H, self.G, self.D, self.V
        q, k, v = q.view(T, G, D), k.view(T, G, D), v.view(T, H, V)
        if self.constant:
            of = torch.arange(H) // (H // G)
            return plain.retention_scan(q[:, of], k[:, of] * 0.6, v, self.decay.double())[0].reshape(T, H * V)
        return plain.state_space_scan(v, k, q, plain.softplus(dt + self.dt_bias.double()), self.a_log.double(), self.skip.double())[0].reshape(T, H * V)

    def step(self, x, lens, contexts, slots):
        """q, k, v and dt lie in the middle of wider rows."""
        ops = _ops()
        H, G, D, V = self.H, self.G, self.D, self.V
        T = x[0].shape[0]
        p = self.pad
        wide = torch.full((T, 2 * G * D + H * V + 4 * p), float("nan"), dtype=self.dt, device=DEV)
        q, k, v = wide[:, p:p + G * D], wide[:, 2 * p + G * D:2 * p + 2 * G * D], wide[:, 3 * p + 2 * G * D:3 * p + 2 * G * D + H * V]
        for dst, src in zip((q, k, v), x):
            dst.copy_(src)
        dtw = torch.full((T, H + 5), float("nan"), device=DEV)
        dtw[:, 3:3 + H] = x[3].to(DEV)
        meta = _meta(list(lens), list(contexts))
        runs = ops.head_decay_chunk_count(meta)
        o = torch.full((T, H * V), float("nan"), device=DEV)
        kw = dict(k_scale=0.6, decay=(self.decay.to(DEV), torch.log2(self.decay.double()).to(DEV))) if self.constant else \
            dict(dt=(dtw[:, 3:3 + H], self.dt_bias.to(DEV), self.a_log.to(DEV)), skip=self.skip.to(DEV))
        if runs:
            kw.update(chunk_states=torch.full((runs, H, D, V), float("nan"), device=DEV), run_numbers=torch.full((runs, H, ops.HEAD_DECAY_RUN), float("nan"), device=DEV))
        ops.head_decay_scan(q, k, v, self.S, meta, torch.tensor(slots, dtype=torch.int32, device=DEV), o, H, G, D, V, **kw)
        return o.cpu()

    def sequence(self, x, cuts, slot):
        outs, pos = [], 0
        for c in cuts:
            outs.append(self.step([t[pos:pos + c] for t in x], [c], [pos + c], [slot]))
            pos += c
        return torch.cat(outs)


def _close(got, ref, rel=3e-6):
    """Relative to the largest value: sums of hundreds of terms of either sign."""
    assert torch.isfinite(got).all()
    err, top = (got.double() - ref).abs().max().item(), ref.abs().max().item()
    assert err <= rel * max(top, 1e-3), (err, top)


SCANS = [(2, 2, 16, 32), (4, 4, 45, 68), (2, 1, 13, 20), (2, 1, 8, 8), (4, 2, 72, 136), (3, 1, 24, 40), (4, 2, 64, 64), (2, 1, 7, 5), (2, 2, 64, 128), (6, 3, 128, 64), (1, 1, 130, 70), (2, 2, 256, 24), (1, 1, 300, 12)]


@both
@pytest.mark.parametrize("constant", [True, False])
@pytest.mark.parametrize("pad", [4, 8])
@pytest.mark.parametrize("H, G, D, V", SCANS)
def test_recurrence_against_the_plain_one_and_cut_anywhere(dtype, constant, pad, H, G, D, V):
    """Rows of bfloat16 that start on 16 bytes (``pad`` 8) run the tensor-core kernels for prompts where the sizes allow."""
    run = _Scan(H, G, D, V, dtype, constant, seed=H * 100 + D)
    run.pad = pad
    x = run.inputs(200, H + D + V)
    ref = run.plain(x)
    whole = run.sequence(x, [200], 1)                                    # three runs of 64 tokens and a rest of 8
    single = run.sequence(x, [1] * 200, 2)
    cut = run.sequence(x, [2, 1, 30, 2, 64, 1, 65, 35], 0)
    for got in (whole, single, cut):
        _close(got, ref)
    ops = _ops()
    ops.head_decay_chunks = False
    try:                                                                 # token by token, a token's arithmetic is the same wherever
        assert torch.equal(run.sequence(x, [200], 1), single)            # the sequence was cut
    finally:
        ops.head_decay_chunks = True


@both
@pytest.mark.parametrize("constant", [True, False])
def test_recurrence_of_unequal_requests_with_slots_used_again(dtype, constant):
    run = _Scan(4, 2, 24, 40, dtype, constant, seed=77, slots=5)
    run.pad = 8
    totals, first = [90, 31, 140, 131, 66], [89, 30, 70, 1, 64]
    xs = [run.inputs(n, 200 + 10 * i) for i, n in enumerate(totals)]
    refs, slots = [run.plain(x) for x in xs], [4, 0, 2, 3, 1]

    def check(order, lo, hi):
        lens = [hi[i] - lo[i] for i in order]
        out = run.step([torch.cat([xs[i][j][lo[i]:hi[i]] for i in order]) for j in range(4)], lens, [hi[i] for i in order], [slots[i] for i in order])
        at = 0
        for i, n in zip(order, lens):
            _close(out[at:at + n], refs[i][lo[i]:hi[i]])
            at += n
    check([3, 0, 1, 2, 4], [0] * 5, first)
    check([0, 1, 4, 2, 3], first, totals)
    out = run.step([torch.cat([xs[2][j][:100], xs[0][j][:65]]) for j in range(4)], [100, 65], [100, 65], [4, 2])      # what the slots held must not show
    _close(out[:100], refs[2][:100])
    _close(out[100:], refs[0][:65])


@both
@pytest.mark.parametrize("a_log, dt_bias", [(6.0, 4.0), (-12.0, 2.0), (0.0, -30.0), (2.0, 60.0), (-3.0, -4.0)])
def test_recurrence_that_forgets_at_once_or_never(dtype, a_log, dt_bias):
    """Decays of 0 in float32, decays so close to 1 that nothing is forgotten, steps of almost nothing and of sixty."""
    run = _Scan(2, 1, 16, 24, dtype, False, a_log=a_log, dt_bias=dt_bias)
    run.pad = 8
    x = run.inputs(150, 9)
    ref = run.plain(x)
    for cuts, slot in (([150], 0), ([1] * 150, 1), ([70, 2, 78], 2)):
        _close(run.sequence(x, cuts, slot), ref, rel=1e-5)


@both
def test_recurrence_a_slow_stretch_behind_strong_decays_keeps_its_digits(dtype):
    """Within one run of 64 tokens the first twenty decay by e^-900 each and the rest hardly at all: differences of large sums of
    logarithms would have lost the digits of the small ones."""
    run = _Scan(1, 1, 8, 16, dtype, False, a_log=4.5, dt_bias=0.0)
    run.pad = 8
    x = run.inputs(64, 4)
    x[3][:20], x[3][20:] = 10.0, -13.0
    x[0][:], x[1][:] = x[0].abs(), x[1].abs()                            # no cancellation in the sums
    ref = run.plain(x)
    got = run.sequence(x, [64], 0)
    rel = ((got[21:].double() - ref[21:]).abs() / ref[21:].abs().clamp(min=1e-6)).median()
    assert rel < 1e-6, rel


@both
@pytest.mark.parametrize("constant", [True, False])
def test_recurrence_carries_the_first_token_across_many_runs(dtype, constant):
    """One channel is written by the first token alone and read by the last one alone."""
    run = _Scan(1, 1, 8, 16, dtype, constant, decay=[1.0], a_log=-25.0, dt_bias=0.5)
    run.pad = 8
    T = 401
    x = run.inputs(T, 22)
    x[1][1:, 3] = 0
    x[1][0, 3] = 2.0
    x[0][T - 1] = 0
    x[0][T - 1, 3] = 1.5
    ref = run.plain(x)
    for cuts in ([T], [300, 101], [400, 1], [1] * T):
        assert torch.allclose(run.sequence(x, cuts, 0)[T - 1].double(), ref[T - 1], atol=1e-5, rtol=1e-5)


# ---- the convolution ----------------------------------------------------------------------------------------
@both
@pytest.mark.parametrize("C, taps", [(24, 4), (40, 2), (64, 3), (21, 4), (21, 6), (300, 4), (32, 1), (16, 5), (520, 7)])
@pytest.mark.parametrize("pad", [4, 5])
def test_convolution_with_bias_and_silu_cut_anywhere(dtype, C, taps, pad):
    ops, dt = _ops(), DT[dtype]
    w, b = torch.randn(C, taps, generator=g(1)), torch.randn(C, generator=g(2))
    state = torch.full((4, max(taps - 1, 1), C), float("nan"), device=DEV)
    tol = dict(atol=2e-6, rtol=1e-5) if dtype == "float32" else dict(atol=1e-2, rtol=1e-2)

    def step(us, lens, contexts, slots):
        u = torch.cat(us)
        wide = torch.full((u.shape[0], C + 2 * pad), float("nan"), device=DEV)
        wide[:, pad:pad + C] = u.to(DEV)
        out = torch.full((u.shape[0], C), float("nan"), dtype=dt, device=DEV)
        ops.conv_silu(wide[:, pad:pad + C], w.to(DEV), b.to(DEV), state[:, :taps - 1].contiguous() if taps == 1 else state, _meta(lens, contexts),
                      torch.tensor(slots, dtype=torch.int32, device=DEV), out)
        return out.float().cpu().double().split(lens)
    us = [torch.randn(n, C, generator=g(10 + n)) for n in (61, 37, 90)]
    refs = [plain.silu(plain.causal_conv(u.double(), w.double(), b.double())) for u in us]
    at, slots = [0, 0, 0], [2, 0, 3]
    for round_ in ([1, 17, 2], [16, 1, 33], [1, 1, 1], [2, 3, 16], [1, 1, 17], [40, 14, 1]):
        round_ = [min(n, u.shape[0] - a) for n, u, a in zip(round_, us, at)]
        order = [i for i in range(3) if round_[i] == 1] + [i for i in range(3) if round_[i] > 1]
        outs = step([us[i][at[i]:at[i] + round_[i]] for i in order], [round_[i] for i in order], [at[i] + round_[i] for i in order], [slots[i] for i in order])
        for i, o in zip(order, outs):
            assert torch.allclose(o, refs[i][at[i]:at[i] + round_[i]], **tol)
            at[i] += round_[i]
    assert torch.allclose(step([us[1]], [37], [37], [2])[0], refs[1], **tol)                # a slot used again


# ---- norms ----------------------------------------------------------------------------------------------------
@both
@pytest.mark.parametrize("gate_first", [True, False])
@pytest.mark.parametrize("W, groups, weighted", [(96, 2, True), (45, 3, False), (512, 1, True), (2048, 2, True), (8192, 1, True), (1024, 16, False), (130, 13, True)])
def test_norm_in_groups_with_a_gate_on_either_side(dtype, gate_first, W, groups, weighted):
    ops, dt, T, eps = _ops(), DT[dtype], 19, 1e-5
    y, z = torch.randn(T, W, generator=g(1)) * torch.linspace(0.1, 4, W), (torch.randn(T, W, generator=g(2)) * 2).to(dt)
    w = torch.rand(W, generator=g(3)) + 0.3 if weighted else None
    f = w.double() if weighted else 1.0
    s = plain.silu(z.double())
    ref = plain.over_rms_in_groups(y.double() * s, groups, eps) * f if gate_first else plain.over_rms_in_groups(y.double(), groups, eps) * f * s
    wide = torch.full((T, W + 8), float("nan"), dtype=dt, device=DEV)
    wide[:, 4:4 + W] = z.to(DEV)
    out = torch.full((T, W + 8), 7.0, dtype=dt, device=DEV)
    ops.gated_group_norm(y.to(DEV), wide[:, 4:4 + W], w.to(DEV) if weighted else None, groups, eps, out[:, 4:4 + W], gate_first)
    tol = dict(atol=2e-5, rtol=1e-5) if dtype == "float32" else dict(atol=3e-2, rtol=1e-2)
    assert torch.allclose(out[:, 4:4 + W].float().cpu().double(), ref, **tol) and (out[:, :4] == 7.0).all() and (out[:, 4 + W:] == 7.0).all()


@both
@pytest.mark.parametrize("W", [40, 53, 1030, 1024, 4096, 9000, 17000])
def test_the_stream_takes_terms_with_scales_and_norms_of_their_own(dtype, W):
    ops, dt, T, eps = _ops(), DT[dtype], 7, 1e-5
    r = lambda s, n=T: torch.randn(n, W, generator=g(W + s)) if n > 1 else torch.randn(W, generator=g(W + s))
    x, ys, scales = r(0), [r(i).to(dt) * (3.0 ** i) for i in (1, 2, 3)], [r(i, 1) for i in (4, 5, 6)]
    va, vb, w = r(7, 1), r(8, 1), r(9, 1)
    tol = dict(atol=2e-5, rtol=2e-5) if dtype == "float32" else dict(atol=3e-2, rtol=1e-2)
    dev = lambda t: t.to(DEV) if t is not None else None

    def joined(terms, vectors):
        s = x.double()
        for y, f, e in terms:
            v = plain.over_rms(y.double(), e) if e is not None else y.double()
            s = s + (v * f.double() if f is not None else v)
        return s + sum(v.double() for v in vectors)
    for terms, vectors in (([(ys[0], scales[0], 1e-5), (ys[1], scales[1], 1e-3), (ys[2], scales[2], None)], [va]),
                           ([(ys[0], scales[0], None), (ys[1], None, None)], [va, vb]), ([(ys[2], None, 1e-6)], []), ([], [])):
        want = joined(terms, vectors)
        res, out = dev(x).clone(), torch.empty(T, W, dtype=dt, device=DEV)
        ops.stream_norm(res, [(dev(y), dev(f), e) for y, f, e in terms], [dev(v) for v in vectors], dev(w), eps, out)
        assert torch.allclose(res.cpu().double(), want, atol=1e-5, rtol=1e-5)
        assert torch.allclose(out.float().cpu().double(), plain.over_rms(want, eps) * w.double(), **tol)
        # a copy of the stream beside other columns
        res, wide = dev(x).clone(), torch.full((T, 2 * W), 7.0, dtype=dt, device=DEV)
        ops.stream_norm(res, [(dev(y), dev(f), e) for y, f, e in terms], [dev(v) for v in vectors], None, 0.0, wide[:, :W])
        assert torch.allclose(res.cpu().double(), want, atol=1e-5, rtol=1e-5) and (wide[:, W:] == 7.0).all()
        assert torch.allclose(wide[:, :W].float().cpu().double(), want, **tol)
        # some rows only, the stream untouched
        rows = torch.tensor([5, 0, 5], dtype=torch.int32)
        res, out = dev(x).clone(), torch.empty(3, W, dtype=dt, device=DEV)
        ops.stream_norm(res, [(dev(y), dev(f), e) for y, f, e in terms], [dev(v) for v in vectors], dev(w), eps, out, rows=dev(rows))
        assert torch.equal(res.cpu(), x)
        assert torch.allclose(out.float().cpu().double(), plain.over_rms(want[rows.long()], eps) * w.double(), **tol)


# ---- the embedding ----------------------------------------------------------------------------------------------
@both
def test_embedding_with_position_rows_and_a_copy(dtype):
    ops, dt, T, V, P, W = _ops(), DT[dtype], 6, 17, 30, 52
    table, pos = torch.randn(V, W, generator=g(1)).to(dt), torch.randn(P, W, generator=g(2)).to(dt)
    ids, at = torch.tensor([3, 0, 16, ~1, 5, 9], dtype=torch.int32), torch.tensor([0, 29, 7, 7, 12, 1], dtype=torch.int32)
    feedback = torch.tensor([4, 11], dtype=torch.int32)
    out, wide, err = torch.empty(T, W, device=DEV), torch.full((T, 2 * W), 7.0, dtype=dt, device=DEV), torch.zeros(4, dtype=torch.int32, device=DEV)
    ops.embed(ids.to(DEV), table.to(DEV), out, err, feedback=feedback.to(DEV), position_rows=(pos.to(DEV), at.to(DEV)), copy=wide[:, W:])
    want = table[[3, 0, 16, 11, 5, 9]].float() + pos[at.long()].float()
    assert torch.equal(out.cpu(), want) and torch.equal(wide[:, W:].cpu(), want.to(dt)) and (wide[:, :W] == 7.0).all() and not err.any()


# ---- attention ------------------------------------------------------------------------------------------------------
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


def _case(dtype, H, G, D, V, ps, window, lens, contexts, seed, boost=None, scale=0.37, sink=True):
    """The attention on requests whose last ``lens`` tokens are this step's queries, with a gate a head and a one in the denominator; (got,
    reference) per request.  Pages wholly behind the first query's window are gone."""
    ops, dt = _ops(), DT[dtype]
    qs = [torch.randn(c, H, D, generator=g(seed + i)) for i, c in enumerate(contexts)]
    ks = [torch.randn(c, G, D, generator=g(seed + 10 + i)) for i, c in enumerate(contexts)]
    vs = [torch.randn(c, G, V, generator=g(seed + 20 + i)) + 2.0 for i, c in enumerate(contexts)]      # (a lost sink shows in the mean)
    if boost:
        boost(qs, ks)
    qs, ks, vs = ([t.to(dt).float() for t in ts] for ts in (qs, ks, vs))       # what the kernel is given, exactly
    row = ops.padded_head(max(D, V))
    pool, bt = _paged(ks, vs, ps, row, dt, seed)
    for b, (n, c) in enumerate(zip(lens, contexts)):
        for i in range((c - n - window + 1) // ps if c - n - window + 1 > 0 else 0):
            pool[bt[b, i]] = float("nan")
            bt[b, i] = -1
    meta = _meta(list(lens), list(contexts))
    T = sum(lens)
    q = torch.zeros(T, H, row)
    q[:, :, :D] = torch.cat([qq[c - n:] for qq, n, c in zip(qs, lens, contexts)])
    gate = torch.full((T, H + 9), float("nan"))
    gate[:, 5:5 + H] = torch.randn(T, H, generator=g(seed + 40)) * 2
    wide = torch.full((T, H * V + 24), 7.0, dtype=dt, device=DEV)              # the results go to columns of a wider tensor
    out = wide[:, 8:8 + H * V]
    ops.sink_attention(q.view(T, -1).to(dt).to(DEV), gate.to(DEV)[:, 5:5 + H], out, pool, ps, bt, meta, H, G, row, V, scale, window, sink,
                       padded=True, gate_heads=True)
    assert not meta.error_flag.any() and (wide[:, :8] == 7.0).all() and (wide[:, 8 + H * V:] == 7.0).all()
    res, at = [], 0
    for qq, kk, vv, n, c in zip(qs, ks, vs, lens, contexts):
        ref = plain.window_attention(qq.double(), kk.double(), vv.double(), scale, window, sink)[c - n:]
        ref = ref * torch.sigmoid(gate[at:at + n, 5:5 + H].double())[:, :, None]
        res.append((out[at:at + n].float().cpu().double(), ref.reshape(n, H * V)))
        at += n
    return res


ATOL, RTOL = {"float32": 2e-5, "bfloat16": 2e-2}, {"float32": 1e-5, "bfloat16": 1e-2}
LENS, CONTEXTS = (1, 1, 1, 70, 45, 2, 150), (1, 97, 300, 70, 211, 130, 150)


@both
@pytest.mark.parametrize("window", [1, 33, 64, 1000])
@pytest.mark.parametrize("H, G, D, V, ps", [(4, 2, 16, 24, 16), (3, 1, 10, 9, 8), (8, 2, 64, 64, 16), (6, 2, 40, 56, 64), (4, 4, 128, 128, 32), (5, 1, 48, 40, 16),
                                            (16, 1, 32, 96, 128), (2, 1, 144, 40, 16)])
def test_windowed_attention_with_a_one_in_the_denominator_and_a_gate_a_head(dtype, H, G, D, V, ps, window):
    for got, ref in _case(dtype, H, G, D, V, ps, window, LENS, CONTEXTS, seed=H * D):
        assert torch.allclose(got, ref, atol=ATOL[dtype], rtol=RTOL[dtype])


@both
@pytest.mark.parametrize("D, ps, window", [(64, 16, 48), (64, 64, 100), (40, 8, 17), (128, 32, 128), (64, 128, 129)])
@pytest.mark.parametrize("distance", [-1, 0])
def test_one_sharp_key_just_inside_or_outside_the_window(dtype, D, ps, window, distance):
    """A key at window - 1 tokens back (seen) or at ``window`` (not) has a score of 40 above the others, for a decoded token and for
    one inside a portion."""
    def boost(qs, ks):
        for r, (qq, kk) in enumerate(zip(qs, ks)):
            p = qq.shape[0] - 1 - 50 * r
            kk[p - window - distance] = qq[p, 0:1] * (40.0 / 0.37) / (qq[p, 0] ** 2).sum()
    for got, ref in _case(dtype, 2, 1, D, D, ps, window, (1, 60), (331, 331), seed=11 + D, boost=boost):
        assert torch.allclose(got, ref, atol=ATOL[dtype], rtol=RTOL[dtype] * 2)


@both
def test_without_strong_scores_the_one_takes_its_share(dtype):
    """All scores far below zero: almost everything goes to the one in the denominator, in prompts and single tokens."""
    def boost(qs, ks):
        for qq, kk in zip(qs, ks):
            qq[:] = qq.abs()
            kk[:] = -kk.abs() * 0.5
    for got, ref in _case(dtype, 2, 1, 64, 64, 16, 40, (1, 60), (100, 90), seed=3, boost=boost, scale=0.4):
        assert ref.mean() < 0.45 and torch.allclose(got, ref, atol=ATOL[dtype], rtol=RTOL[dtype])
    for got, ref in _case(dtype, 2, 1, 64, 64, 16, 40, (1, 60), (100, 90), seed=3, boost=boost, scale=0.4, sink=False):
        assert ref.mean() > 0.7 and torch.allclose(got, ref, atol=ATOL[dtype], rtol=RTOL[dtype])


@both
@pytest.mark.parametrize("H, G, D, V, rot", [(4, 2, 8, 24, 6), (3, 3, 10, 9, 10), (4, 1, 64, 64, 32), (1, 1, 80, 96, 2), (16, 4, 64, 64, 64), (8, 8, 120, 40, 120)])
@pytest.mark.parametrize("T, extra", [(37, 5), (139, 8)])
def test_bias_weighted_norm_and_yarn_rotation_into_the_cache(dtype, H, G, D, V, rot, T, extra):
    from mini_engine_b200.parts import FrequencyRotary
    ops, dt, ps, eps = _ops(), DT[dtype], 8, 1e-5
    scaling = {"factor": 6.0, "original": 200, "fast": 12.0, "slow": 1.0}
    C = H * D + G * (D + V)
    proj, b = torch.randn(T, C + extra, generator=g(1)) * 2, torch.randn(C, generator=g(2))
    qw, kw = torch.rand(D, generator=g(3)) + 0.3, torch.rand(D, generator=g(4)) + 0.3
    positions = torch.tensor([0, 1, 2, 3, 70001, 1 << 20] + list(range(500, 500 + T - 6)), dtype=torch.int32)
    x = proj[:, :C].double() + b.double()
    freqs, magnitude = plain.yarn_frequencies(rot, 3000.0, scaling)
    q = plain.over_rms(x[:, :H * D].view(T, H, D), eps) * qw.double()
    k = plain.over_rms(x[:, H * D:(H + G) * D].view(T, G, D), eps) * kw.double()
    q, k = plain.rotate_halves(q, positions, freqs, magnitude), plain.rotate_halves(k, positions, freqs, magnitude)
    rope = FrequencyRotary(rot, 3000.0, scaling)
    rope.finalize(torch.float32, DEV)
    row = ops.padded_head(max(D, V))
    pool = torch.full((20, 2, G, ps, row), float("nan"), dtype=dt, device=DEV)
    slots = torch.randperm(20 * ps, generator=g(5))[:T].to(torch.int32)
    q_out = torch.full((T, H * row), float("nan"), dtype=dt, device=DEV)
    ops.attn_prep(proj.to(DEV), b.to(DEV), qw.to(DEV), kw.to(DEV), "before", eps, rope.freq, positions.to(DEV), slots.to(DEV), q_out, pool, ps, H, G, D, V,
                  magnitude=rope.magnitude)
    tol = dict(atol=3e-5, rtol=1e-5) if dtype == "float32" else dict(atol=3e-2, rtol=1e-2)
    got = q_out.float().cpu().double().view(T, H, row)
    assert torch.allclose(got[..., :D], q, **tol) and (got[..., D:] == 0).all()
    rows = pool.float().cpu().double()
    for t in range(T):
        page, off = int(slots[t]) // ps, int(slots[t]) % ps
        assert torch.allclose(rows[page, 0, :, off, :D], k[t], **tol) and (rows[page, 0, :, off, D:] == 0).all()
        assert torch.allclose(rows[page, 1, :, off, :V], x[t, (H + G) * D:].view(G, V), **tol) and (rows[page, 1, :, off, V:] == 0).all()


# ---- the router and the experts ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("E, top, groups, keep, scale", [(8, 3, 4, 2, 0.7), (6, 2, 3, 1, 1.3), (5, 2, 5, 3, 2.0), (12, 4, 1, 1, 1.0), (64, 6, 8, 3, 1.5), (4, 4, 2, 2, 0.5),
                                                         (130, 2, 2, 1, 1.0)])
@pytest.mark.parametrize("T", [1, 21, 90])
def test_routing_by_softmax_over_groups(E, top, groups, keep, scale, T):
    """Short steps route and sort in one kernel, long ones in three; the logits are columns of wider rows."""
    ops = _ops()
    z = torch.full((T, E + 3), float("nan"))
    z[:, :E] = torch.randn(T, E, generator=g(E + T)) * 3
    idx, wgt = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    counts, offsets = torch.empty(E, dtype=torch.int32, device=DEV), torch.empty(E + 1, dtype=torch.int32, device=DEV)
    order, place = torch.empty(T * top, dtype=torch.int32, device=DEV), torch.empty(T * top, dtype=torch.int32, device=DEV)
    ops.moe_route_grouped_sort(z.to(DEV)[:, :E], None, top, groups, keep, idx, wgt, counts, offsets, order, place, softmax=True, scale=scale)
    seen = [0] * E
    for t in range(T):
        chosen, w = plain.route(z[t, :E].double(), top, groups, keep, scale)
        assert idx[t].tolist() == chosen
        assert torch.allclose(wgt[t].cpu().double(), torch.stack(w), rtol=1e-5, atol=1e-9)
        for e in chosen:
            seen[e] += 1
    assert offsets.tolist() == [0] + np.cumsum(seen).tolist()
    flat = idx.view(-1)[order.long()].tolist()
    assert flat == sorted(flat) and order[place.long()].tolist() == list(range(T * top))


@both
@pytest.mark.parametrize("T, W, F, S", [(1, 64, 40, 24), (9, 52, 22, 30), (40, 128, 64, 96), (300, 128, 72, 128)])
@pytest.mark.parametrize("shared", [True, False])
def test_experts_with_a_gated_shared_one(dtype, T, W, F, S, shared):
    from mini_engine_b200.parts import RoutedExperts
    dt, E, top = DT[dtype], 6, 2
    ff = RoutedExperts(W, E, top, F, router_bias=False, routing="softmax_groups", groups=(3, 2), activation="relu_squared", weight_scale=1.4,
                       shared={"intermediate_size": S, "activation": "relu_squared"} if shared else None, shared_gate="shared.sg" if shared else None)
    w = {"router": torch.randn(E, W, generator=g(1)) * (4 / W ** 0.5)}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = torch.randn(F, W, generator=g(10 + e)) * (1.5 / W ** 0.5), torch.randn(W, F, generator=g(30 + e)) / F ** 0.5
    if shared:
        w["shared.up"], w["shared.down"] = torch.randn(S, W, generator=g(50)) * (1.5 / W ** 0.5), torch.randn(W, S, generator=g(51)) / S ** 0.5
        w["shared.sg"] = torch.randn(1, W, generator=g(52)) * (2 / W ** 0.5)
    w = {k: v.to(dt) for k, v in w.items()}
    ff.router.params["router"] = torch.cat([w["router"]] + ([w["shared.sg"]] if shared else [])).to(DEV)
    ff.params["experts_gate_up"] = torch.cat([w[f"e{e}.up"] for e in range(E)]).to(DEV)
    ff.params["experts_down"] = torch.cat([w[f"e{e}.down"] for e in range(E)]).to(DEV)
    if shared:
        ff.shared.up.params["up"], ff.shared.down.params["down"] = w["shared.up"].to(DEV), w["shared.down"].to(DEV)
    ff.finalize(dt, DEV)
    x = torch.randn(T, W, generator=g(3)).to(dt)
    ctx = SimpleNamespace(act_dtype=dt, error_flag=torch.zeros(4, dtype=torch.int32, device=DEV),
                          buffer=lambda name, shape, dtype, zero=False: torch.zeros(shape, dtype=dtype, device=DEV))
    got = ff.forward(x.to(DEV), ctx).float().cpu().double()
    assert not ctx.error_flag.any()
    cfg = {"router": {"experts": E, "top": top, "scale": 1.4, "groups": {"count": 3, "keep": 2}}, "shared": shared}
    ref = plain.routed_experts(x.double(), {k: v.double() for k, v in w.items()}, "", cfg)
    tol = dict(atol=2e-5, rtol=1e-4) if dtype == "float32" else dict(atol=1e-1, rtol=2e-2)
    assert torch.allclose(got, ref, **tol)
