"""GPU tests of the Goluzen design in the layered family against the NumPy oracle tests/goluzen_ref.py: the new kernels alone (the
seam of residual add and norm, the epilogues of products, the sigmoid router with group limits, gated linear attention in its
one-token and its chunked form, attention with everything the design puts into one layer, latent attention with direct queries and
a window), then whole models under every schedule the step function admits, and greedy generation through the scheduler and the
command line.  Configurations are small and random; where random weights would hide a fault (a key at a window's edge, the last
kept first position, a far key among hundreds, a sink, a state carried over many tokens) the inputs are made so that it decides
the answer.  float32 mode is held to 2e-4."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import pygpukit_b200 as gk
from pygpukit_b200 import llm
from pygpukit_b200._lib import api
from pygpukit_b200.llm.config import layered_config_from_json
from pygpukit_b200.llm.layers.linear import LinearRows
from pygpukit_b200.llm.paged_cache import PagedKVCache
from tests import goluzen_ref as R

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_KEEP = []


def keep(g):
    """Park a device array until the test ends (kernels run asynchronously)."""
    _KEEP.append(g)
    return g


@pytest.fixture(autouse=True)
def _release_parked_arrays():
    yield
    gk.synchronize()
    _KEEP.clear()


def i32(a):
    return keep(gk.from_numpy(np.ascontiguousarray(a, np.int32)))


def f32(a):
    return keep(gk.from_numpy(np.ascontiguousarray(a, np.float32)))


def f64(a):
    return keep(gk.from_numpy(np.ascontiguousarray(a, np.float64)))


def mat(a, dtype):
    if dtype == "float32":
        return f32(a)
    return keep(gk.from_numpy((np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)))


def cuts_of(sizes):
    at = [0]
    for n in sizes:
        at.append(at[-1] + n)
    return list(zip(at, at[1:]))


# ================================================================ kernels alone
@pytest.mark.parametrize("rows", [3, 40])
@pytest.mark.parametrize("W,top", [(5, 1), (40, 3), (301, 0), (2048, 6), (5003, 2), (16384, 1), (256, 70)])
def test_residual_add_and_next_norm_in_one_launch(W, top, rows):
    rng = np.random.default_rng(W + top)
    x, base, shared, w = (rng.standard_normal(n) for n in ((rows, W), (rows, W), (rows, W), W))
    parts, inv, wt = rng.standard_normal((max(1, rows * top), W)), rng.permutation(max(1, rows * top)), rng.uniform(0, 1, max(1, rows * top))
    gate = rng.standard_normal((rows, 4))
    experts = (wt[:, None] * parts[inv]).reshape(rows, top, W).sum(1) if top else 0.0
    P, I, T, B, S, G, Wd = f32(parts), i32(inv), f32(wt), f32(base), f32(shared), f32(gate), f32(w)
    h = keep(gk.zeros((rows, W), gk.float32))
    for use_base, use_parts, use_shared, use_gate, use_h in ((0, 0, 0, 0, 1), (1, 0, 0, 0, 1), (0, 1, 0, 0, 1), (0, 1, 1, 1, 1), (1, 1, 1, 0, 1), (1, 1, 1, 1, 0)):
        use_parts = use_parts and top > 0
        d = f32(x)
        api.rms_add_norm_f32(B.device_ptr if use_base else None, P.device_ptr if use_parts else None, I.device_ptr if use_parts else None,
                             T.device_ptr if use_parts else None, top if use_parts else 0, S.device_ptr if use_shared else None,
                             G.device_ptr if use_gate else None, 4, 2, d.device_ptr, Wd.device_ptr, 1.0, 1e-5,
                             h.device_ptr if use_h else None, rows, W, None)
        want = x + (base if use_base else 0) + (experts if use_parts else 0)
        if use_shared:
            want = want + (R.sigmoid(gate[:, 2:3]) if use_gate else 1.0) * shared
        assert np.abs(d.to_numpy() - want).max() < 3e-5
        if use_h:
            assert np.abs(h.to_numpy() - R.unit_rms(want, 1e-5) * (1.0 + w)).max() < 3e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [1, 7, 70])
def test_activation_and_gate_epilogues_of_the_products(rows, dtype):
    rng = np.random.default_rng(rows)
    K, F, H, Dv = 50, 37, 3, 7
    x, up = R.bf16_round(rng.standard_normal((rows, K))), R.bf16_round(rng.standard_normal((F, K)) / 5)
    out, xd, z = keep(gk.zeros((rows, F), gk.float32)), f32(x), x.astype(np.float64) @ up.T
    for epi, act in ((6, R.relu2), (9, R.gelu_tanh)):
        p = LinearRows(mat(up, dtype), epilogue=epi)
        for product in (p.forward, p.forward_seq):
            product(xd.device_ptr, K, rows, out.device_ptr, F)
            assert np.abs(out.to_numpy() - act(z)).max() < 1e-4 * np.abs(act(z)).max()
    # one product per head on a slice of the row, times the sigmoid of the same columns of wider gate rows
    w, gate = R.bf16_round(rng.standard_normal((H, Dv, 10))), rng.standard_normal((rows, H * Dv + 9))
    out, gd = keep(gk.zeros((rows, H * Dv), gk.float32)), f32(gate)
    LinearRows(mat(w, dtype)).forward_seq(xd.device_ptr, K, rows, out.device_ptr, H * Dv, epilogue=10, batch=H, a_batch=10, c_batch=Dv,
                                          aux=(gd.device_ptr, 0, None, H * Dv + 9, 4))
    want = np.concatenate([x[:, 10 * h:10 * h + 10].astype(np.float64) @ w[h].T for h in range(H)], axis=1) * R.sigmoid(gate[:, 4:4 + H * Dv])
    assert np.abs(out.to_numpy() - want).max() < 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_squared_relu_experts_grouped_and_row_by_row(dtype):
    rng = np.random.default_rng(3)
    E, F, K, T = 5, 11, 24, 60
    w, x = R.bf16_round(rng.standard_normal((E, F, K))), R.bf16_round(rng.standard_normal((T, K)))
    p, xd = LinearRows(mat(w, dtype), epilogue=6), f32(x)
    of = np.array([0, 2, 3, 1, 4, 2, 0, 3])
    out = keep(gk.zeros((T, F), gk.float32))
    p.forward_per_row(xd.device_ptr, K, 8, out.device_ptr, F, None, i32(of).device_ptr)
    want = np.stack([R.relu2(x[i].astype(np.float64) @ w[e].T) for i, e in enumerate(of)])
    assert np.abs(out.to_numpy()[:8] - want).max() < 1e-4 * want.max()
    off, perm = [0, 20, 20, 21, 47, 60], rng.permutation(T)                  # an expert without rows, one with a single row
    p.forward_grouped(xd.device_ptr, K, out.device_ptr, F, i32(perm).device_ptr, i32(off).device_ptr, T)
    want = np.concatenate([R.relu2(x[perm[a:b]].astype(np.float64) @ w[e].T) for e, (a, b) in enumerate(zip(off, off[1:]))])
    assert np.abs(out.to_numpy() - want).max() < 1e-4 * want.max()


@pytest.mark.parametrize("E,top,count,keep_groups,extra", [(12, 3, 4, 2, False), (8, 2, 2, 1, True), (6, 1, 6, 3, True), (70, 33, 7, 5, False),
                                                           (9, 4, 1, 1, True), (10, 2, 5, 5, False), (64, 8, 8, 1, True), (1, 1, 1, 1, True)])
@pytest.mark.parametrize("shift", [0.0, -4.0])
def test_sigmoid_router_with_group_limits(E, top, count, keep_groups, extra, shift):
    """shift: corrections that make every choice score negative (an expert outside the kept groups must still lose)"""
    rng = np.random.default_rng(E * 7 + top)
    T, slots = 37, top + extra
    z, bias = (2 * rng.standard_normal((T, E + 2))).astype(np.float32), (rng.uniform(-1, 1, E) + shift).astype(np.float32)
    idx, wt = i32(np.zeros(T * slots)), f32(np.zeros(T * slots))
    rank, counts = i32(np.zeros(T * slots)), i32(np.zeros(E + 1))
    zd, bd = f32(z), f32(bias)
    api.moe_route_sigmoid(zd.device_ptr, E + 2, T, E, top, bd.device_ptr, count, keep_groups, 2.25, E if extra else -1, idx.device_ptr,
                          wt.device_ptr, rank.device_ptr, counts.device_ptr, None)
    order, w = R.route(z[:, :E].astype(np.float64), bias.astype(np.float64), top, count, keep_groups, 2.25)
    if extra:
        order, w = np.concatenate([order, np.full((T, 1), E)], 1), np.concatenate([w, R.sigmoid(z[:, E:E + 1].astype(np.float64))], 1)
    got = idx.to_numpy().reshape(T, slots)
    assert (got == order).all() and np.abs(wt.to_numpy().reshape(T, slots) - w).max() < 1e-5
    assert (counts.to_numpy() == np.bincount(order.reshape(-1), minlength=E + 1)).all()
    r = rank.to_numpy().reshape(-1)
    for e in range(E + 1):                                               # the ranks of an expert's rows are 0 .. count - 1
        assert sorted(r[got.reshape(-1) == e]) == list(range(int((order == e).sum())))


class DecayHarness:
    """Gated linear attention on raw rows [q | k | v | gate | y]: pgk_seq_gla_step, or pgk_seq_gla_decays / _chunks (and the finish
    launch for wide values)."""

    def __init__(self, H, D, Dv, inner=5, tau=4.0, slots=3, seg=0, pad=0):
        self.H, self.D, self.Dv, self.r, self.tau, self.seg = H, D, Dv, inner, tau, seg
        rng = np.random.default_rng(H * 13 + D)
        self.state = f32(7.0 * np.ones((slots, H * D * Dv)))             # dirty
        self.w2, self.b2 = 2 * rng.standard_normal((H * D, inner)) / np.sqrt(inner), rng.uniform(-2.0, 4.0, H * D)
        self.w = 1 + 0.2 * rng.standard_normal(Dv)
        self.pos = {}
        self.cols = 2 * H * D + 2 * H * Dv + inner + pad

    def random_rows(self, T, seed):
        return np.random.default_rng(seed).standard_normal((T, self.cols))

    def run(self, batch, chunked=False):
        """batch: [(slot, rows [n, cols])] -> [n, H * Dv] per entry"""
        H, D, Dv = self.H, self.D, self.Dv
        rows = np.concatenate([r for _, r in batch])
        seqs, row = [], 0
        for s, r in batch:
            p0 = self.pos.get(s, 0)
            seqs.append((row, len(r), s, p0))
            self.pos[s] = p0 + len(r)
            row += len(r)
        T, longest = len(rows), max(len(r) for _, r in batch)
        proj, out = f32(rows), keep(gk.zeros((T, H * Dv), gk.float32))
        k_off, v_off, g_off = H * D, 2 * H * D, 2 * H * D + H * Dv
        y_off = g_off + H * Dv
        sq, w2, b2, w = i32(seqs), f32(self.w2.T), f32(self.b2), f32(np.tile(self.w, H))
        S = self.state.device_ptr
        if longest == 1 and not chunked:
            api.seq_gla_step(proj.device_ptr, self.cols, 0, k_off, v_off, g_off, y_off, self.r, w2.device_ptr, b2.device_ptr, 1.0 / self.tau,
                             D ** -0.5, w.device_ptr, 1e-6, out.device_ptr, H * Dv, S, sq.device_ptr, len(seqs), H, D, Dv, None)
        else:
            nch = -(-longest // api.seq_gla_chunk_tokens(D, Dv))
            seg = min(self.seg or nch, nch)
            sums, ws = keep(gk.zeros((T * H * D,), gk.float32)), f32(5.0 * np.ones(len(seqs) * seg * H * D * (Dv + 1)))
            api.seq_gla_decays(proj.device_ptr, self.cols, y_off, self.r, w2.device_ptr, b2.device_ptr, 1.0 / self.tau, sq.device_ptr, len(seqs),
                               longest, H, D, sums.device_ptr, None)
            for c0 in range(0, nch, seg):
                api.seq_gla_chunks(proj.device_ptr, self.cols, 0, k_off, v_off, g_off, sums.device_ptr, D ** -0.5, w.device_ptr, 1e-6,
                                   out.device_ptr, H * Dv, S, sq.device_ptr, len(seqs), H, D, Dv, c0, min(seg, nch - c0), ws.device_ptr, None)
            if not api.seq_gla_fused_finish(Dv):
                api.seq_linear_finish(out.device_ptr, H * Dv, proj.device_ptr, self.cols, g_off, w.device_ptr, T, H, Dv, 1, 2, 1e-6, 1.0, None)
        o, at, res = out.to_numpy(), 0, []
        for _, r in batch:
            res.append(o[at:at + len(r)])
            at += len(r)
        return res

    def oracle(self, rows):
        H, D, Dv, T = self.H, self.D, self.Dv, len(rows)
        q, k = rows[:, :H * D].reshape(T, H, D) * D ** -0.5, rows[:, H * D:2 * H * D].reshape(T, H, D)
        v, g = (rows[:, 2 * H * D + j * H * Dv:2 * H * D + (j + 1) * H * Dv] for j in (0, 1))
        y = rows[:, 2 * H * D + 2 * H * Dv:2 * H * D + 2 * H * Dv + self.r]
        a = R.sigmoid(y @ self.w2.T + self.b2) ** (1.0 / self.tau)
        o = R.decayed_recurrence(q, k, v.reshape(T, H, Dv), a.reshape(T, H, D))
        return (R.unit_rms(o, 1e-6) * self.w).reshape(T, H * Dv) * R.silu(g)


# key sizes that fill chunks of 64, 32 and 16 tokens, values of one column, of one block and of several
DECAY_LAYOUTS = [dict(H=3, D=8, Dv=6), dict(H=1, D=44, Dv=60, tau=16.0, pad=3), dict(H=2, D=70, Dv=9, inner=1), dict(H=2, D=130, Dv=20, tau=1.0),
                 dict(H=5, D=16, Dv=33, inner=40), dict(H=2, D=20, Dv=260), dict(H=1, D=12, Dv=1030), dict(H=4, D=64, Dv=128, inner=16),
                 dict(H=2, D=1, Dv=1), dict(H=1, D=300, Dv=12, tau=30.0), dict(H=1, D=600, Dv=8, inner=3)]


@pytest.mark.parametrize("layout", DECAY_LAYOUTS)
def test_gated_linear_attention_whole_portions_and_single_tokens_agree_with_the_oracle(layout):
    h = DecayHarness(**layout)
    T = 150
    rows = h.random_rows(T, h.D)
    ref = h.oracle(rows)
    for s, sizes in enumerate([[T], [2] * 10 + [33, 1, 1, 64, 31], [1] * 70 + [80], [63, 1, 65, 21], [16, 17, 15, 48, 54]]):
        got = np.concatenate([h.run([(s % 3, rows[a:b])])[0] for a, b in cuts_of(sizes)])
        assert np.abs(got - ref).max() < 5e-5 * max(1.0, np.abs(ref).max()), sizes
        h.pos.pop(s % 3)                                                 # the slot is used again from position 0, state dirty


def test_chunk_sizes_follow_the_key_size():
    assert [api.seq_gla_chunk_tokens(D, 64) for D in (16, 128, 300, 600)] == [64, 64, 32, 16]
    assert api.seq_gla_chunk_tokens(5000, 64) == 0


@pytest.mark.parametrize("seg", [1, 2, 3])
def test_gated_linear_attention_in_segments_of_chunks(seg):
    h = DecayHarness(2, 24, 20, seg=seg)
    a, b = h.random_rows(330, 1), h.random_rows(100, 2)                  # the second sequence has fewer chunks than the first
    ra, rb = h.oracle(a), h.oracle(b)
    x, y = h.run([(0, a[:300]), (1, b[:70])])
    assert np.abs(x - ra[:300]).max() < 5e-5 and np.abs(y - rb[:70]).max() < 5e-5
    x, y = h.run([(0, a[300:]), (1, b[70:])])
    assert np.abs(x - ra[300:]).max() < 5e-5 and np.abs(y - rb[70:]).max() < 5e-5


def test_gated_linear_attention_single_tokens_through_the_chunked_form():
    h = DecayHarness(3, 10, 14)
    rows = h.random_rows(12, 3)
    got = np.concatenate([h.run([(1, rows[t:t + 1])], chunked=t % 2 == 0)[0] for t in range(12)])
    assert np.abs(got - h.oracle(rows)).max() < 5e-5


def test_gated_linear_attention_unequal_sequences_in_one_step():
    h = DecayHarness(2, 12, 10)
    data = [h.random_rows(n, n) for n in (140, 3, 17)]
    refs = [h.oracle(d) for d in data]
    cut = (130, 1, 9)
    first = h.run([(s, d[:n]) for s, (d, n) in enumerate(zip(data, cut))])
    rest = [[] for _ in data]
    for j in range(10):                                                  # then token by token, sequences ending at different steps
        live = [s for s, (d, n) in enumerate(zip(data, cut)) if n + j < len(d)]
        for s, o in zip(live, h.run([(s, data[s][cut[s] + j:cut[s] + j + 1]) for s in live])):
            rest[s].append(o)
    for a, b, r in zip(first, rest, refs):
        assert np.abs(np.concatenate([a] + b) - r).max() < 5e-5


@pytest.mark.parametrize("decoded", [False, True])
def test_one_early_token_is_carried_over_hundreds_on_the_channel_that_keeps_it(decoded):
    """Channel 0 never decays and only one token writes on it; channel 1 halves with every token: hundreds of tokens later the query
    on both reads the early value alone."""
    H, D, Dv, T, star = 2, 16, 12, 330, 4
    h = DecayHarness(H, D, Dv, tau=1.0)
    h.w2[:] = 0.0
    b = np.full((H, D), 0.0)
    b[:, 0] = 60.0                                                       # sigmoid(60): everything is kept
    h.b2 = b.reshape(-1)
    rng = np.random.default_rng(1)
    rows = h.random_rows(T, 5)
    q, k = np.zeros((T, H, D)), 0.3 * rng.standard_normal((T, H, D))
    q[:, :, 0] = q[:, :, 1] = 5.0
    k[:, :, 0] = k[:, :, 1] = 0.0
    k[star, :, 0], k[star, :, 1] = 4.0, 4.0
    rows[:, :H * D], rows[:, H * D:2 * H * D] = q.reshape(T, -1), k.reshape(T, -1)
    ref = h.oracle(rows)
    sizes = [star + 2] + [1] * (T - star - 2) if decoded else [100, 130, 100]
    got = np.concatenate([h.run([(0, rows[a:b])])[0] for a, b in cuts_of(sizes)])
    assert np.abs(got - ref).max() < 5e-5
    v = rows[star, 2 * H * D:2 * H * D + H * Dv].reshape(H, Dv)
    want = (R.unit_rms(v, 1e-6) * h.w).reshape(-1) * R.silu(rows[:, 2 * H * D + H * Dv:2 * H * D + 2 * H * Dv])
    assert np.abs(got[star:] - want[star:]).max() < 1e-3 and np.abs(got[:star]).max() < 1e-6


@pytest.mark.parametrize("low,high", [(-300.0, -200.0), (-40.0, 40.0), (30.0, 90.0), (-8.0, -4.0)])
def test_gated_linear_attention_with_decays_at_their_extremes(low, high):
    """States forgotten within a token, kept for good, and both beside each other in one head: no exponent may leave its range, and
    strong decays must not wash out the weights of the tokens behind them."""
    h = DecayHarness(2, 10, 8, tau=1.0)
    h.b2 = np.random.default_rng(2).uniform(low, high, 20)
    rows = h.random_rows(200, 11)
    ref = h.oracle(rows)
    got = np.concatenate([h.run([(0, rows[a:b])])[0] for a, b in cuts_of([1, 2, 130] + [1] * 40 + [27])])
    assert np.isfinite(got).all() and np.abs(got - ref).max() < 1e-4 * max(1.0, np.abs(ref).max())


class AttentionHarness:
    """pgk_seq_mixer_prep_rot_ex2 + pgk_seq_attention_ex3 on raw rows [q | k | v] with biases, half-layout rotation with a position
    factor, unit-norm q / k behind it, tanh cap, window with kept first positions and a sink per head."""

    def __init__(self, H, G, D, Dv, window, first, scale=0.3, cap=5.0, page=4, dims=0, base=50.0, factor=3.0, splits=1, norm=True, sinks=True,
                 biases=True):
        self.H, self.G, self.D, self.Dv, self.window, self.first, self.scale, self.cap, self.splits = H, G, D, Dv, window, first, scale, cap, splits
        self.dims, self.norm = dims, norm
        self.cache = PagedKVCache([(G, D, Dv)], "float32", page, 64, 2)
        self.qt = api.seq_queries_per_tile(H, G)
        rng = np.random.default_rng(H * 31 + D)
        self.rot = {"dims": dims, "base": base, "scaling": {"factor": factor}}
        self.bias = [rng.standard_normal(n) if biases else np.zeros(n) for n in (H * D, G * D, G * Dv)]
        self.sinks = rng.uniform(-1, 3, H) if sinks else None
        self.inv_freq = f64(R.plain_frequencies(self.rot)) if dims else None
        self.tickets = gk.zeros((4096,), gk.int32)
        self.cols = H * D + G * D + G * Dv

    def run(self, seq, q, k, v):
        n = q.shape[0]
        slot, pos0 = self.cache.extend(seq, n)
        self.cache.sync_table()
        c, H, G, D, Dv = self.cache, self.H, self.G, self.D, self.Dv
        proj = f32(np.concatenate([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], axis=1))
        single = 1 if n == 1 and pos0 > 0 else 0
        b = [f32(x) for x in self.bias]
        api.seq_mixer_prep_rot_ex2(proj.device_ptr, self.cols, n, H, G, D, Dv, 0, H * D, H * D + G * D, self.dims,
                                   self.inv_freq.device_ptr if self.dims else None, 1 if self.norm else 0, None, None, 1e-6, b[0].device_ptr,
                                   b[1].device_ptr, b[2].device_ptr, None, 0, 0, None, 0, 0, None, None, single, c.k[0].device_ptr,
                                   c.v[0].device_ptr, c.dtype_code, c.table_dev.device_ptr, c.pool.max_pages, c.page_size,
                                   i32([slot] * n).device_ptr, i32(np.arange(pos0, pos0 + n)).device_ptr, None)
        tiles = [(i, min(self.qt, n - i), slot, pos0 + i) for i in range(0, n, self.qt)]
        out = keep(gk.zeros((n, H * Dv), gk.float32))
        api.seq_attention_ex3(proj.device_ptr, self.cols, 0, None, 0, 0, 0, out.device_ptr, H * Dv, c.k[0].device_ptr,
                              c.v[0].device_ptr, D, Dv, c.dtype_code, c.table_dev.device_ptr, c.pool.max_pages, c.page_size,
                              i32(tiles).device_ptr, len(tiles), None, None, f32(self.sinks).device_ptr if self.sinks is not None else None,
                              H, G, D, Dv, 0, self.window, self.first, self.scale, self.cap, 0, None, 1.0, 0, 0, None, None, None, 0,
                              self.splits, keep(gk.zeros((n * H * self.splits * (Dv + 2),), gk.float32)).device_ptr,
                              self.tickets.device_ptr, single, None)
        return out.to_numpy().reshape(n, H, Dv)

    def oracle(self, q, k, v):
        q, k, v = (x + b.reshape(x.shape[1:]) for x, b in zip((q, k, v), self.bias))
        if self.dims:
            f, p = R.plain_frequencies(self.rot), np.arange(len(q))
            q, k = R.rotate(q, p, f, False), R.rotate(k, p, f, False)
        if self.norm:
            q, k = R.unit_rms(q, 1e-6), R.unit_rms(k, 1e-6)
        return R.softmax_attention(q, k, v, self.scale, self.cap, self.window, self.first, self.sinks)


# windows of one, beyond the sequence and none; more kept positions than the window holds, than a page holds, one, none
ATTENTION_LAYOUTS = [dict(H=4, G=2, D=16, Dv=8, window=7, first=3, dims=8), dict(H=6, G=2, D=8, Dv=12, window=3, first=5, dims=8, page=3),
                     dict(H=3, G=3, D=12, Dv=20, window=100, first=4, dims=4), dict(H=2, G=1, D=40, Dv=72, window=20, first=33, dims=12, page=8),
                     dict(H=1, G=1, D=6, Dv=70, window=1, first=1, dims=2), dict(H=2, G=2, D=10, Dv=10, window=0, first=0, dims=10),
                     dict(H=4, G=1, D=8, Dv=130, window=5, first=0, dims=6, page=2, cap=0.0), dict(H=40, G=1, D=8, Dv=6, window=6, first=2, dims=2, page=16, sinks=False),
                     dict(H=2, G=2, D=9, Dv=7, window=4, first=3, dims=4, factor=1.0, biases=False)]


@pytest.mark.parametrize("layout", ATTENTION_LAYOUTS)
def test_attention_agrees_with_the_oracle(layout):
    h = AttentionHarness(**layout)
    rng = np.random.default_rng(h.H * 7 + h.D)
    T = 75
    q, k, v = 3 * rng.standard_normal((T, h.H, h.D)), 3 * rng.standard_normal((T, h.G, h.D)), rng.standard_normal((T, h.G, h.Dv))
    ref = h.oracle(q, k, v)
    for name, sizes in (("whole", [T]), ("portions", [2, 2, 9, 1, 17, 14, 30]), ("decoded", [5] + [1] * 70), ("from zero", [1] * 30 + [45])):
        got = np.concatenate([h.run(name, q[a:b], k[a:b], v[a:b]) for a, b in cuts_of(sizes)])
        assert np.abs(got - ref).max() < 3e-5, name
        h.cache.release(name)                                            # the next one inherits its pages


@pytest.mark.parametrize("splits", [2, 3, 7])
@pytest.mark.parametrize("n_last", [1, 6])
def test_attention_in_key_slices_counts_the_sink_once(splits, n_last):
    h = AttentionHarness(4, 2, 12, 14, window=200, first=5, dims=8, page=8, splits=splits)
    h.sinks = np.array([4.0, -2.0, 6.0, 0.0])
    rng = np.random.default_rng(splits)
    T = 400
    q, k, v = rng.standard_normal((T, 4, 12)), rng.standard_normal((T, 2, 12)), rng.standard_normal((T, 2, 14))
    h.run("a", q[:T - n_last], k[:T - n_last], v[:T - n_last])
    got = h.run("a", q[T - n_last:], k[T - n_last:], v[T - n_last:])
    assert np.abs(got - h.oracle(q, k, v)[T - n_last:]).max() < 3e-5


def standout(T, H, G, D, Dv, star):
    """inputs whose token `star` outweighs all others in every score, with a value that tells"""
    rng = np.random.default_rng(star)
    q, k = np.zeros((T, H, D)), 0.1 * rng.standard_normal((T, G, D))
    q[:, :, 4] = 10.0
    k[:, :, 4] = -1.0
    k[star, 0, 4] = 2.0
    v = 0.01 * rng.standard_normal((T, G, Dv))
    v[star, 0, 1] = 1.0
    return q, k, v


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("window,first,page", [(9, 3, 4), (64, 4, 16), (65, 5, 64), (6, 17, 4), (130, 1, 64)])
def test_standout_token_at_the_window_edge_and_at_the_last_kept_position(window, first, page, decoded):
    H, G, D, Dv = 2, 1, 8, 4
    for star in sorted({0, first - 1, first, first + 1, page - 1, page, 2 * page + 1}):
        T = star + window + 4
        q, k, v = standout(T, H, G, D, Dv, star)
        h = AttentionHarness(H, G, D, Dv, window, first, scale=1.0, cap=30.0, page=page, dims=4, norm=False, sinks=False, biases=False)
        n0 = star + 1 if decoded else T - 3
        got = np.concatenate([h.run("a", q[:n0], k[:n0], v[:n0])] + [h.run("a", q[i:i + 1], k[i:i + 1], v[i:i + 1]) for i in range(n0, T)])
        assert np.abs(got - h.oracle(q, k, v)).max() < 1e-4
        for i in range(T):
            assert np.abs(got[i, :, 1] - (1.0 if i >= star and (i - star < window or star < first) else 0.0)).max() < 0.1, (star, i)


@pytest.mark.parametrize("decoded", [False, True])
def test_far_key_among_hundreds(decoded):
    H, G, D, Dv, page, T = 1, 1, 4, 2, 8, 600
    for star in (0, 7, 8, 300, 587):
        q, k, v = np.zeros((T, H, D)), np.zeros((T, G, D)), np.zeros((T, G, Dv))
        q[:, :, 0], k[star, :, 0] = 6.0, 6.0
        v[:, :, 0] = 0.01 * np.arange(T)[:, None]
        h = AttentionHarness(H, G, D, Dv, 0, 0, scale=1.0, cap=0.0, page=page, norm=False, sinks=False, biases=False)
        n0 = T - 5 if decoded else T
        out = [h.run("a", q[:n0], k[:n0], v[:n0])] + [h.run("a", q[i:i + 1], k[i:i + 1], v[i:i + 1]) for i in range(n0, T)]
        assert np.abs(np.concatenate(out)[-5:, 0, 0] - 0.01 * star).max() < 1e-4, star


@pytest.mark.parametrize("decoded", [False, True])
def test_sink_that_outweighs_every_key_and_the_cap_that_does_not_touch_it(decoded):
    """Scores capped at 5 against a sink of 12: what is left of a value is about T exp(5 - 12); a sink that were capped, scaled or
    counted twice gives another number."""
    h = AttentionHarness(2, 1, 8, 4, window=6, first=2, scale=50.0, cap=5.0, dims=4, biases=False)
    h.sinks = np.array([12.0, -12.0])
    T = 30
    q, k, v = np.ones((T, 2, 8)), np.ones((T, 1, 8)), np.ones((T, 1, 4))
    ref = h.oracle(q, k, v)
    got = np.concatenate([h.run("a", q[a:b], k[a:b], v[a:b]) for a, b in cuts_of([5] + [1] * 25 if decoded else [T])])
    assert np.abs(got - ref).max() < 1e-6 and np.abs(got[:, 1] - 1.0).max() < 1e-4 and 1e-3 < got[-1, 0, 0] < 0.02


class LatentHarness:
    """pgk_seq_latent_prep_heads + pgk_seq_attention_ex on raw rows [q heads (plain | rotated) | c', r'], the queries taken as absorbed
    already (plain size = latent size)."""

    def __init__(self, H, R_, Dr, window, scale=0.3, page=4, rot=None, splits=1):
        self.H, self.R, self.Dr, self.window, self.scale, self.splits = H, R_, Dr, window, scale, splits
        self.rot = rot or {"dims": Dr, "base": 90.0, "scaling": {"factor": 3.0, "original": 40, "fast": 4.0, "slow": 1.0}}
        self.freq, self.mult = R.stretched_frequencies(self.rot) if Dr else (np.zeros(1), 1.0)
        self.cache = PagedKVCache([(1, R_ + Dr, 0)], "float32", page, 64, 2)
        self.qt = api.seq_queries_per_tile(H, 1)
        self.w = np.random.default_rng(R_).uniform(0.5, 1.5, R_)
        self.inv_freq, self.tickets = f64(self.freq), gk.zeros((4096,), gk.int32)

    def run(self, seq, q, y):
        n, H, L, Dr = q.shape[0], self.H, self.R, self.Dr
        slot, pos0 = self.cache.extend(seq, n)
        self.cache.sync_table()
        c, row, cols = self.cache, L + Dr, H * (L + Dr) + L + Dr
        proj, qa = f32(np.concatenate([q.reshape(n, -1), y], axis=1)), f32(q.reshape(n, -1))
        qa_tail = q.copy()
        qa_tail[..., L:] = 99.0                                          # the launch puts the turned tails there
        qa = f32(qa_tail.reshape(n, -1))
        pos, w = i32(np.arange(pos0, pos0 + n)), f32(self.w)
        api.seq_latent_prep_heads(proj.device_ptr, cols, n, row, L, H, qa.device_ptr, H * row, row, L, H * row, L, Dr, self.rot["dims"] if Dr else 0,
                                  w.device_ptr, 0.0, 1e-6, self.inv_freq.device_ptr, self.mult, c.k[0].device_ptr, c.dtype_code,
                                  c.table_dev.device_ptr, c.pool.max_pages, c.page_size, i32([slot] * n).device_ptr, pos.device_ptr, None)
        tiles = [(i, min(self.qt, n - i), slot, pos0 + i) for i in range(0, n, self.qt)]
        out = keep(gk.zeros((n, H * L), gk.float32))
        api.seq_attention_ex(qa.device_ptr, H * row, 0, None, 0, 0, 0, out.device_ptr, H * L, c.k[0].device_ptr, c.k[0].device_ptr, row, row,
                             c.dtype_code, c.table_dev.device_ptr, c.pool.max_pages, c.page_size, i32(tiles).device_ptr, len(tiles), None, None,
                             H, 1, row, L, 0, self.window, self.scale, 0.0, self.splits,
                             keep(gk.zeros((n * H * self.splits * (L + 2),), gk.float32)).device_ptr, self.tickets.device_ptr,
                             1 if n == 1 and pos0 > 0 else 0, None)
        return out.to_numpy().reshape(n, H, L)

    def oracle(self, q, y):
        L, p = self.R, np.arange(len(q))
        c, r = R.unit_rms(y[:, :L], 1e-6) * self.w, y[:, None, L:]
        tail = q[..., L:]
        if self.Dr:
            r, tail = R.rotate(r, p, self.freq, True, self.mult), R.rotate(tail, p, self.freq, True, self.mult)
        k = np.concatenate([c[:, None], r], axis=-1)
        return R.softmax_attention(np.concatenate([q[..., :L], tail], axis=-1), k, c[:, None], self.scale, window=self.window)


LATENT_LAYOUTS = [dict(H=3, R_=14, Dr=8, window=7), dict(H=1, R_=5, Dr=2, window=1), dict(H=5, R_=40, Dr=16, window=0, page=8),
                  dict(H=33, R_=9, Dr=4, window=20, page=16), dict(H=2, R_=264, Dr=10, window=30), dict(H=2, R_=12, Dr=0, window=5, page=3),
                  dict(H=2, R_=8, Dr=12, window=9, rot={"dims": 6, "base": 30.0}), dict(H=6, R_=130, Dr=30, window=64, page=64)]


@pytest.mark.parametrize("layout", LATENT_LAYOUTS)
def test_latent_rows_window_and_scaled_rotation_agree_with_the_oracle(layout):
    h = LatentHarness(**layout)
    rng = np.random.default_rng(h.H + h.R)
    T = 75
    q, y = rng.standard_normal((T, h.H, h.R + h.Dr)), rng.standard_normal((T, h.R + h.Dr))
    ref = h.oracle(q, y)
    for name, sizes in (("whole", [T]), ("portions", [2, 2, 9, 1, 17, 14, 30]), ("decoded", [5] + [1] * 70)):
        got = np.concatenate([h.run(name, q[a:b], y[a:b]) for a, b in cuts_of(sizes)])
        assert np.abs(got - ref).max() < 3e-5, name
        h.cache.release(name)


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("window,page,splits", [(9, 4, 1), (64, 16, 2), (65, 64, 1), (130, 64, 3)])
def test_standout_latent_at_the_window_edge(window, page, splits, decoded):
    L = 6
    for star in (0, page - 1, page, 2 * page + 1):
        T = star + window + 4
        q, y = np.zeros((T, 2, L)), np.zeros((T, L))
        y[:, 0] = 1.0                                                    # every latent is [2.4, 0, ..], the standout [0, 2.4, ..]
        y[star] = [0, 1, 0, 0, 0, 0]
        q[:, :, 1] = 12.0
        h = LatentHarness(2, L, 0, window, scale=1.0, page=page, splits=splits)
        h.w[:] = 1.0
        n0 = star + 1 if decoded else T - 3
        got = np.concatenate([h.run("a", q[:n0], y[:n0])] + [h.run("a", q[i:i + 1], y[i:i + 1]) for i in range(n0, T)])
        assert np.abs(got - h.oracle(q, y)).max() < 1e-4
        for i in range(T):
            assert (got[i, :, 1] > 2.0).all() == (0 <= i - star < window), (star, i)


# ================================================================ whole models
def variants():
    """Sizes that the mechanisms must not assume equal or 1: key and value sizes, head counts, rotated dimensions below the head
    size and equal to it, windows of one, beyond the sequence and none, kept positions in any relation to them, no cap, no position
    scaling, one latent read by two layers with windows and head counts of their own, one chosen expert and all of them, one group,
    groups of one, shared experts narrower, as wide and wider than the others and none, layers without feed-forward, odd widths,
    every order of layers, values wider than one block's columns."""
    yield "base", R.make_config([R.latent_layer(mlp=R.dense_ff()), R.gla_layer(mlp=R.moe_ff()), R.attention_layer(mlp=R.moe_ff(shared_ff=12)),
                                 R.latent_layer(kv_from=0, mlp=R.moe_ff(shared_ff=20))])
    yield "attention_first", R.make_config([R.attention_layer(heads=6, kv_heads=3, dim=10, vdim=4, dims=10, window=5, keep_first=7, softcap=2.0, factor=1.0, mlp=R.moe_ff(top=1, groups=(2, 1), shared_ff=0)),
                                            R.gla_layer(heads=2, dim=5, vdim=9, tau=1.0, mlp=R.dense_ff(31)), R.latent_layer(heads=5, dim=3, rot_dim=6, vdim=11, kv_rank=7, window=1, scale=0.9),
                                            R.attention_layer(heads=2, kv_heads=1, dim=16, vdim=20, dims=2, window=1, keep_first=1, mlp=R.moe_ff(experts=8, top=4, groups=(4, 2), scale=0.3))],
                                           vocab=61, width=52, embed_scale=0.7)
    yield "shared_latents", R.make_config([R.gla_layer(heads=1, dim=70, vdim=140, mlp=R.moe_ff(experts=3, top=3, ff=8, groups=None, shared_ff=8)),
                                           R.latent_layer(heads=2, window=9), R.latent_layer(heads=4, dim=6, vdim=5, window=30, kv_from=1, scale=0.7, mlp=R.dense_ff(7)),
                                           R.attention_layer(heads=3, kv_heads=3, dim=6, vdim=6, dims=4, window=1000, keep_first=2),
                                           R.latent_layer(heads=1, dim=20, vdim=9, window=2, kv_from=1), R.latent_layer(heads=2, kv_rank=30, rot_dim=4, window=0)], width=33, vocab=47)
    yield "only_attention", R.make_config([R.attention_layer(window=0, keep_first=0, softcap=0.0, mlp=R.moe_ff(experts=40, top=20, ff=5, shared_ff=3, groups=(8, 5))),
                                           R.attention_layer(heads=5, kv_heads=5, window=16, base=1e4, mlp=R.moe_ff(experts=5, top=3, groups=(5, 4)))])
    yield "only_states", R.make_config([R.gla_layer(tau=16.0), R.gla_layer(heads=4, dim=8, vdim=8, tau=2.0, mlp=R.dense_ff(16))])


VARIANTS = dict(variants())


def make(name, dtype="float32", page=4, seed=1, tokens_hint=64, slots=2):
    cfg = json.loads(json.dumps(VARIANTS[name]))
    P = R.random_params(cfg, seed=seed)
    m = llm.build_layered_model(layered_config_from_json(cfg), P, dtype)
    m.init_cache(tokens_hint, page_size=page, slots=slots)
    return cfg, P, m


def tokens(cfg, n, seed=0):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


@pytest.mark.parametrize("name", list(VARIANTS))
def test_whole_prompt_and_every_layer_match_the_oracle_float32(name):
    cfg, P, m = make(name, tokens_hint=128)
    toks = tokens(cfg, 75)
    ref, layers = R.forward(cfg, P, toks, True)
    seen = []
    m.trace_hook = lambda run, x: seen.append(x)
    got = m.step([("a", toks, list(range(len(toks))))])
    assert len(seen) == len(layers)
    for run, (a, b) in enumerate(zip(seen, layers)):
        assert np.abs(a - b).max() < F32_TOL, run
    assert np.abs(got - ref).max() < F32_TOL


@pytest.mark.parametrize("name", list(VARIANTS))
def test_prefill_then_token_by_token_decoding(name):
    cfg, P, m = make(name)
    toks = tokens(cfg, 50, seed=3)
    ref = R.forward(cfg, P, toks)
    got = [m.step([("a", toks[:9], list(range(9)))])]
    got += [m.step([("a", [t], [0])]) for t in toks[9:]]                 # windows pass over decoded tokens
    assert np.abs(np.concatenate(got) - ref).max() < F32_TOL


@pytest.mark.parametrize("name", list(VARIANTS))
def test_first_tokens_and_decoding_from_position_zero(name):
    cfg, P, m = make(name)
    toks = tokens(cfg, 14, seed=4)
    ref = R.forward(cfg, P, toks)
    got = np.concatenate([m.step([("a", [t], [0])]) for t in toks])
    assert np.abs(got - ref).max() < F32_TOL


@pytest.mark.parametrize("sizes", [[2] * 20, [3, 2, 7, 1, 11, 6, 10], [16, 24], [1, 39], [33, 3, 4], [70, 2, 68]])
@pytest.mark.parametrize("name", ["base", "attention_first"])
def test_prompt_portions(name, sizes):
    cfg, P, m = make(name)
    toks = tokens(cfg, sum(sizes), seed=5)
    ref = R.forward(cfg, P, toks)
    got, at = [], 0
    for n in sizes:
        got.append(m.step([("a", toks[at:at + n], list(range(n)))]))
        at += n
    assert np.abs(np.concatenate(got) - ref).max() < F32_TOL


@pytest.mark.parametrize("name", ["base", "attention_first", "shared_latents"])
def test_batch_of_unequal_requests_equals_each_alone(name):
    cfg, P, m = make(name, tokens_hint=16)                               # small pool: pages and slots (with state) grow
    lens, new = [1, 23, 7, 40], 6
    seqs = [tokens(cfg, n + new, seed=10 + i) for i, n in enumerate(lens)]
    refs = [R.forward(cfg, P, s) for s in seqs]
    got = m.step([(i, s[:n], list(range(n))) for i, (s, n) in enumerate(zip(seqs, lens))])
    assert np.abs(got - np.concatenate([r[:n] for r, n in zip(refs, lens)])).max() < F32_TOL
    for j in range(new):                                                 # request 0 ends after two more tokens
        live = [i for i in range(4) if i != 0 or j < 2]
        got = m.step([(i, [seqs[i][lens[i] + j]], [0]) for i in live], end=[0] if j == 1 else [])
        assert np.abs(got - np.stack([refs[i][lens[i] + j] for i in live])).max() < F32_TOL
    assert m.cache.pool.live_sequences == 3


def test_prompts_and_decoded_tokens_in_one_step():
    cfg, P, m = make("base", tokens_hint=128)
    a, b, c = tokens(cfg, 30, seed=1), tokens(cfg, 25, seed=2), tokens(cfg, 9, seed=3)
    ra, rb, rc = (R.forward(cfg, P, s) for s in (a, b, c))
    m.step([("a", a[:20], [])])
    got = m.step([("a", [a[20]], [0]), ("b", b[:24], [0, 23]), ("c", c[:1], [0])])
    assert np.abs(got - np.stack([ra[20], rb[0], rb[23], rc[0]])).max() < F32_TOL
    got = m.step([("c", c[1:], [0, 7]), ("b", [b[24]], [0]), ("a", a[21:], [8])])
    assert np.abs(got - np.stack([rc[1], rc[8], rb[24], ra[29]])).max() < F32_TOL


def test_more_than_eight_decoding_requests():
    cfg, P, m = make("base", tokens_hint=256)
    seqs = [tokens(cfg, 5 + i, seed=30 + i) for i in range(11)]
    refs = [R.forward(cfg, P, s) for s in seqs]
    m.step([(i, s[:-2], []) for i, s in enumerate(seqs)])
    for back in (2, 1):
        got = m.step([(i, [s[-back]], [0]) for i, s in enumerate(seqs)])
        assert np.abs(got - np.stack([r[-back] for r in refs])).max() < F32_TOL


def test_pages_slots_and_state_are_used_again():
    cfg, P, m = make("base", page=4)
    a, b, c = tokens(cfg, 39, seed=20), tokens(cfg, 14, seed=21), tokens(cfg, 42, seed=22)
    m.step([("a", a, []), ("b", b[:6], [])])
    pages_a, slot_a = m.cache.pool.page_list("a"), m.cache.pool.slot("a")
    m.step([("b", b[6:], [])], end=["a"])
    got = m.step([("c", c[:13], list(range(13)))])                       # c inherits a's slot (dirty state) and pages
    assert m.cache.pool.slot("c") == slot_a and set(m.cache.pool.page_list("c")) <= set(pages_a)
    got = np.concatenate([got] + [m.step([("c", [t], [0]), ("b", [1], [])])[:1] for t in c[13:]])
    assert np.abs(got - R.forward(cfg, P, c)).max() < F32_TOL
    m.release("c")
    got = np.concatenate([m.step([("d", [t], [0]), ("b", [2], [])])[:1] for t in c[:16]])     # and a sequence decoded from 0 in it
    assert np.abs(got - R.forward(cfg, P, c[:16])).max() < F32_TOL


def test_layers_that_read_another_layers_latent_have_no_cache_of_their_own():
    cfg, P, m = make("shared_latents")
    assert [k is not None for k in m.cache.k] == [False, True, False, True, False, True] and all(v is None for i, v in enumerate(m.cache.v) if i != 3)


def test_long_decoding_and_wanted_places_subset():
    cfg, P, m = make("base", page=8)
    toks = tokens(cfg, 190, seed=6)
    ref = R.forward(cfg, P, toks)
    want = [0, 6, 7, 8, 30, 69]
    got = m.step([("a", toks[:70], want)])
    assert np.abs(got - ref[want]).max() < F32_TOL
    got = np.concatenate([m.step([("a", [t], [0])]) for t in toks[70:]])
    assert np.abs(got - ref[70:]).max() < F32_TOL


def test_eager_decoding_equals_graph_replay():
    cfg, P, m = make("base", page=8)
    toks = tokens(cfg, 40, seed=9)
    m.step([("a", toks[:10], [])])
    graphed = np.concatenate([m.step([("a", [t], [0])]) for t in toks[10:]])
    m.release("a")
    m.use_graphs = False
    m.step([("b", toks[:10], [])])
    eager = np.concatenate([m.step([("b", [t], [0])]) for t in toks[10:]])
    assert np.array_equal(graphed, eager)


@pytest.mark.parametrize("name", list(VARIANTS))
def test_bfloat16_mode_stays_within_bfloat16_rounding(name):
    cfg, P, m = make(name, dtype="bfloat16")
    toks = tokens(cfg, 40, seed=7)
    ref = R.forward(cfg, P, toks)
    whole = m.step([("a", toks, list(range(40)))])
    scale = np.sqrt(np.mean(ref ** 2))
    assert np.sqrt(np.mean((whole - ref) ** 2)) < 0.05 * scale
    got = np.concatenate([m.step([("b", toks[:20], list(range(20)))])] + [m.step([("b", [t], [0])]) for t in toks[20:]])
    assert np.sqrt(np.mean((got - whole) ** 2)) < 0.05 * scale           # the same sequence cut differently: rounding only


def test_a_sequence_with_state_cannot_be_cut_back_and_one_without_can():
    cfg, P, m = make("base")
    m.step([("a", tokens(cfg, 9), [])])
    with pytest.raises(ValueError, match="cut back"):
        m.cache.truncate("a", 5)
    cfg, P, m = make("only_attention")
    toks = tokens(cfg, 50, seed=2)
    m.step([("a", toks[:33] + [(t + 1) % cfg["vocab"] for t in toks[33:]], [])])
    m.cache.truncate("a", 33)
    got = m.step([("a", toks[33:], list(range(17)))])
    assert np.abs(got - R.forward(cfg, P, toks)[33:]).max() < F32_TOL


def test_greedy_generation_through_the_scheduler():
    cfg, P, m = make("base", tokens_hint=256)
    prompts = [tokens(cfg, n, seed=40 + n) for n in (3, 17, 9)]
    outs = m.generate(prompts, max_new_tokens=12, temperature=0.0, prefill_chunk=5)
    for p, o in zip(prompts, outs):
        assert o[:len(p)] == p and len(o) == len(p) + 12
        seq = list(p)
        for t in o[len(p):]:
            z = R.forward(cfg, P, seq)[-1]
            top2 = np.sort(z)[-2:]
            if top2[1] - top2[0] < 1e-3:                                 # a near tie: either token is right, stop comparing
                break
            assert t == int(np.argmax(z))
            seq.append(t)
    assert m.cache.pool.live_sequences == 0 and m.generate(prompts[0], 2) == outs[0][:len(prompts[0]) + 2]


def test_random_model_of_the_design_runs_in_bfloat16():
    cfg = layered_config_from_json(R.make_config([R.latent_layer(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, window=20, mlp=R.dense_ff(128)),
                                                  R.gla_layer(heads=4, dim=32, vdim=64, mlp=R.moe_ff(experts=4, top=2, ff=64, shared_ff=96, groups=(2, 1))),
                                                  R.attention_layer(heads=4, kv_heads=2, dim=32, vdim=32, dims=16, window=20, mlp=R.moe_ff(experts=4, top=2, ff=64, shared_ff=64, groups=None)),
                                                  R.latent_layer(heads=2, dim=32, rot_dim=16, vdim=32, kv_rank=64, window=9, kv_from=0)], vocab=256, width=128))
    m = llm.random_layered_model(cfg, "bfloat16", seed=3)
    m.init_cache(256)
    toks = tokens({"vocab": 256}, 60)
    whole = m.step([("a", toks, [58, 59])])
    m.step([("b", toks[:59], [])])
    one = m.step([("b", toks[59:], [0])])
    assert np.isfinite(whole).all() and np.abs(one - whole[1:]).max() < 0.05 * np.abs(whole).max()


def _save(cfg, P, folder):
    tensors = {k: ((np.ascontiguousarray(v, np.float32).view(np.uint32) >> 16).astype(np.uint16).reshape(v.shape), "BF16")
               for k, v in P.items()}
    llm.save_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    return {k: (np.ascontiguousarray(v, np.float32).view(np.uint32) >> 16 << 16).view(np.float32) for k, v in P.items()}


def test_loader_picks_the_family_from_config_json(tmp_path):
    cfg = VARIANTS["attention_first"]
    P = _save(cfg, R.random_params(cfg, seed=8), str(tmp_path))
    m = llm.load_model_from_safetensors(str(tmp_path), dtype="float32")
    assert isinstance(m, llm.LayeredCausalModel) and m.config.architecture == "Goluzen"
    toks = tokens(cfg, 30)
    assert np.abs(m.step([("a", toks, list(range(30)))]) - R.forward(cfg, P, toks)).max() < F32_TOL
    with pytest.raises(ValueError, match="shape"):
        bad = dict(P)
        bad["l0.mix.sink"] = P["l0.mix.sink"][:-1]
        llm.build_layered_model(layered_config_from_json(cfg), bad, "float32")


def test_trace_replay_command_line(tmp_path):
    cfg = VARIANTS["base"]
    model_dir, out_dir = tmp_path / "model", tmp_path / "out"
    model_dir.mkdir()
    P = _save(cfg, R.random_params(cfg, seed=9), str(model_dir))
    a, b = tokens(cfg, 24, seed=1), tokens(cfg, 6, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:21], "want": [0, 20]}, {"id": "b", "tokens": b[:5], "want": [4]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[21]], "want": []}, {"id": "b", "tokens": [b[5]], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[22]], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": [a[23]], "want": [0]}], "end": ["a"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(model_dir), "--dtype", "float32",
                        "--out", str(out_dir), "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    ra, rb = R.forward(cfg, P, a), R.forward(cfg, P, b)
    V = cfg["vocab"]
    got0 = np.fromfile(out_dir / "0.f32", "<f4").reshape(-1, V)
    assert np.abs(got0 - np.stack([ra[0], ra[20], rb[4]])).max() < F32_TOL
    assert np.abs(np.fromfile(out_dir / "1.f32", "<f4").reshape(-1, V) - rb[5:6]).max() < F32_TOL
    assert np.abs(np.fromfile(out_dir / "3.f32", "<f4").reshape(-1, V) - ra[23:24]).max() < F32_TOL
