"""GPU tests of the Vosolorn design in the layered family against the NumPy oracle tests/vosolorn_ref.py: the new kernels alone
(the RMS join behind a sublayer, the two gelu epilogues, the logit router, the matrix memory with exponential gates in its
one-token and its chunked form, attention with pooled blocks, a norm in front of a rotation in pairs and rotated values), then
whole models under every schedule the step function admits, and greedy generation through the scheduler and the command line.
Configurations are small and random; where random weights would hide a fault (a key at a window's or a block's edge, a far
block among hundreds, a state carried over many tokens) the inputs are made so that it decides the answer.  float32 mode is
held to 2e-4."""
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
from pygpukit_b200.llm.layers.linear import LinearRows, interleave_gate_up
from pygpukit_b200.llm.paged_cache import PagedKVCache
from tests import vosolorn_ref as R

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


def cuts_of(sizes):
    at = [0]
    for n in sizes:
        at.append(at[-1] + n)
    return list(zip(at, at[1:]))


# ================================================================ kernels alone
@pytest.mark.parametrize("W", [5, 40, 301, 2048, 5003, 16384])
@pytest.mark.parametrize("rows", [3, 40])
def test_rms_join_of_plain_rows(W, rows):
    rng = np.random.default_rng(W)
    x, y, w = rng.standard_normal((rows, W)), 3 * rng.standard_normal((rows, W)), rng.standard_normal(W)
    d = f32(x)
    api.rms_join_f32(f32(y).device_ptr, None, None, None, 0, f32(w).device_ptr, 1e-5, d.device_ptr, rows, W, None)
    assert np.abs(d.to_numpy() - (x + R.unit_rms(y, 1e-5) * w)).max() < 2e-5


@pytest.mark.parametrize("W,top,shared", [(40, 3, True), (33, 1, False), (256, 70, True), (1030, 5, False)])
def test_rms_join_of_weighted_expert_rows(W, top, shared):
    rng = np.random.default_rng(W + top)
    T = 13
    x, base, w = rng.standard_normal((T, W)), rng.standard_normal((T, W)), rng.standard_normal(W)
    parts, inv, wt = rng.standard_normal((T * top, W)), rng.permutation(T * top), rng.uniform(0, 1, T * top)
    d = f32(x)
    api.rms_join_f32(f32(base).device_ptr if shared else None, f32(parts).device_ptr, i32(inv).device_ptr, f32(wt).device_ptr, top,
                     f32(w).device_ptr, 1e-6, d.device_ptr, T, W, None)
    y = (wt[:, None] * parts[inv]).reshape(T, top, W).sum(1) + (base if shared else 0)
    assert np.abs(d.to_numpy() - (x + R.unit_rms(y, 1e-6) * w)).max() < 2e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [1, 7, 70])
def test_gelu_epilogues_of_the_products(rows, dtype):
    rng = np.random.default_rng(rows)
    K, F = 50, 37
    x, gate, up = R.bf16_round(rng.standard_normal((rows, K))), R.bf16_round(rng.standard_normal((F, K))), R.bf16_round(rng.standard_normal((F, K)))

    def mat(a):
        if dtype == "float32":
            return f32(a)
        return keep(gk.from_numpy((np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)))

    out = keep(gk.zeros((rows, F), gk.float32))
    pair, one = LinearRows(mat(interleave_gate_up(gate, up)), epilogue=7), LinearRows(mat(up), epilogue=8)
    assert pair.out_cols == F and one.out_cols == F
    xd = f32(x)
    for product in (lambda p: p.forward(xd.device_ptr, K, rows, out.device_ptr, F),
                    lambda p: p.forward_seq(xd.device_ptr, K, rows, out.device_ptr, F)):
        product(pair)
        want = R.gelu_tanh(x.astype(np.float64) @ gate.T) * (x.astype(np.float64) @ up.T)
        assert np.abs(out.to_numpy() - want).max() < 1e-4 * np.abs(want).max()
        product(one)
        want = R.gelu_erf(x.astype(np.float64) @ up.T)
        assert np.abs(out.to_numpy() - want).max() < 1e-4 * np.abs(want).max()


@pytest.mark.parametrize("E,top,extra", [(10, 3, -1), (5, 1, 5), (70, 40, 70), (4, 4, -1), (1, 1, 1), (33, 2, 33)])
def test_router_that_chooses_and_weighs_by_its_logits(E, top, extra):
    rng = np.random.default_rng(E * 7 + top)
    T, slots = 37, top + (extra >= 0)
    z, bias = 4 * rng.standard_normal((T, E + 2)), rng.standard_normal(E)
    z[0, :E] -= 500.0                                                    # far from zero: only differences count
    idx, wt = i32(np.zeros(T * slots)), f32(np.zeros(T * slots))
    rank, counts = i32(np.zeros(T * slots)), i32(np.zeros(E + 1))
    zd, bd = f32(z), f32(bias)
    api.moe_route_logits(zd.device_ptr, E + 2, T, E, top, bd.device_ptr, extra, idx.device_ptr, wt.device_ptr, rank.device_ptr,
                         counts.device_ptr, None)
    order, w = R.route(z[:, :E].astype(np.float32).astype(np.float64) + bias.astype(np.float32), top)
    if extra >= 0:
        order, w = np.concatenate([order, np.full((T, 1), extra)], 1), np.concatenate([w, np.ones((T, 1))], 1)
    got_i = idx.to_numpy().reshape(T, slots)
    assert (got_i == order).all() and np.abs(wt.to_numpy().reshape(T, slots) - w).max() < 1e-5
    assert (counts.to_numpy() == np.bincount(order.reshape(-1), minlength=E + 1)).all()
    r = rank.to_numpy().reshape(-1)
    for e in range(E + 1):                                               # the ranks of an expert's rows are 0 .. count - 1
        assert sorted(r[got_i.reshape(-1) == e]) == list(range(int((order == e).sum())))
    api.moe_route_logits(zd.device_ptr, E + 2, T, E, top, None, -1, idx.device_ptr, wt.device_ptr, None, None, None)
    order, w = R.route(z[:, :E].astype(np.float32).astype(np.float64), top)
    assert (idx.to_numpy()[:T * top].reshape(T, top) == order).all()


class MemoryHarness:
    """The matrix memory on raw rows [q | k | v | gate | i | f]: pgk_seq_mlstm_step, or pgk_seq_mlstm_gates / _chunks (and the
    finish launch for wide values)."""

    def __init__(self, H, D, Dv, cap=9.0, slots=3, seg=0):
        self.H, self.D, self.Dv, self.cap, self.seg = H, D, Dv, cap, seg
        rng = np.random.default_rng(H * 13 + D)
        self.state = [f32(7.0 * np.ones((slots, n))) for n in (H * D * Dv, H * D, H)]      # dirty
        self.ib, self.fb = rng.standard_normal(H), rng.uniform(1.0, 4.0, H)
        self.w = 1 + 0.2 * rng.standard_normal(H * Dv)
        self.pos = {}
        self.cols = 2 * H * D + 2 * H * Dv + 2 * H

    def random_rows(self, T, seed):
        rng = np.random.default_rng(seed)
        rows = rng.standard_normal((T, self.cols))
        rows[:, -2 * self.H:-self.H] *= 3.0                              # input gates far apart
        return rows

    def run(self, batch, chunked=None):
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
        g_off = 2 * H * D + H * Dv
        S, N, M = (a.device_ptr for a in self.state)
        sq = i32(seqs)
        ib, fb, w = f32(self.ib), f32(self.fb), f32(self.w)
        args = (proj.device_ptr, self.cols, 0, H * D, 2 * H * D, g_off, g_off + H * Dv, g_off + H * Dv + H, ib.device_ptr,
                fb.device_ptr, self.cap, D ** -0.5, w.device_ptr, 1e-6, out.device_ptr, H * Dv, S, N, M, sq.device_ptr, len(seqs))
        if longest == 1 and not chunked:
            api.seq_mlstm_step(*args, H, D, Dv, None)
        else:
            MC = api.seq_mlstm_chunk_tokens()
            nch = -(-longest // MC)
            seg = min(self.seg or nch, nch)
            gates = keep(gk.zeros((api.seq_mlstm_gate_floats(T, H),), gk.float32))
            ws = f32(5.0 * np.ones(len(seqs) * seg * H * D * (Dv + 1)))
            api.seq_mlstm_gates(proj.device_ptr, self.cols, g_off + H * Dv, g_off + H * Dv + H, ib.device_ptr, fb.device_ptr,
                                self.cap, M, sq.device_ptr, len(seqs), T, H, gates.device_ptr, None)
            for c0 in range(0, nch, seg):
                api.seq_mlstm_chunks(*args, T, H, D, Dv, gates.device_ptr, c0, min(seg, nch - c0), ws.device_ptr, None)
            if not api.seq_mlstm_fused_finish(Dv):
                api.seq_linear_finish(out.device_ptr, H * Dv, proj.device_ptr, self.cols, g_off, w.device_ptr, T, H, Dv, 1, 1, 1e-6,
                                      1.0, None)
        o, at, res = out.to_numpy(), 0, []
        for _, r in batch:
            res.append(o[at:at + len(r)])
            at += len(r)
        return res

    def oracle(self, rows):
        H, D, Dv, T = self.H, self.D, self.Dv, len(rows)
        q, k = rows[:, :H * D].reshape(T, H, D) * D ** -0.5, rows[:, H * D:2 * H * D].reshape(T, H, D)
        v, g = (rows[:, 2 * H * D + j * H * Dv:2 * H * D + (j + 1) * H * Dv] for j in (0, 1))
        i = self.cap * np.tanh((rows[:, -2 * H:-H] + self.ib) / self.cap)
        f = R.log_sigmoid(self.cap * np.tanh((rows[:, -H:] + self.fb) / self.cap))
        o = R.unit_rms(R.mlstm_recurrence(q, k, v.reshape(T, H, Dv), i, f), 1e-6).reshape(T, H * Dv)
        return o * self.w * R.sigmoid(g)


MEMORY_LAYOUTS = [dict(H=3, D=8, Dv=6), dict(H=1, D=44, Dv=60, cap=2.0), dict(H=2, D=70, Dv=9), dict(H=2, D=130, Dv=20, cap=40.0),
                  dict(H=5, D=16, Dv=33), dict(H=2, D=20, Dv=260), dict(H=1, D=12, Dv=1030), dict(H=4, D=64, Dv=128), dict(H=2, D=1, Dv=1)]


@pytest.mark.parametrize("layout", MEMORY_LAYOUTS)
def test_matrix_memory_whole_portions_and_single_tokens_agree_with_the_oracle(layout):
    h = MemoryHarness(**layout)
    T = 150
    rows = h.random_rows(T, h.D)
    ref = h.oracle(rows)
    for s, sizes in enumerate([[T], [2] * 10 + [33, 1, 1, 64, 31], [1] * 70 + [80], [63, 1, 65, 21]]):
        got = np.concatenate([h.run([(s % 3, rows[a:b])])[0] for a, b in cuts_of(sizes)])
        assert np.abs(got - ref).max() < 5e-5, sizes
        h.pos.pop(s % 3)                                                 # the slot is used again from position 0, state dirty


@pytest.mark.parametrize("seg", [1, 2, 3])
def test_matrix_memory_in_segments_of_chunks(seg):
    h = MemoryHarness(2, 24, 20, seg=seg)
    a, b = h.random_rows(330, 1), h.random_rows(100, 2)                  # the second sequence has fewer chunks than the first
    ra, rb = h.oracle(a), h.oracle(b)
    x, y = h.run([(0, a[:300]), (1, b[:70])])
    assert np.abs(x - ra[:300]).max() < 5e-5 and np.abs(y - rb[:70]).max() < 5e-5
    x, y = h.run([(0, a[300:]), (1, b[70:])])
    assert np.abs(x - ra[300:]).max() < 5e-5 and np.abs(y - rb[70:]).max() < 5e-5


def test_matrix_memory_single_tokens_through_the_chunked_form():
    h = MemoryHarness(3, 10, 14)
    rows = h.random_rows(12, 3)
    got = np.concatenate([h.run([(1, rows[t:t + 1])], chunked=t % 2 == 0)[0] for t in range(12)])
    assert np.abs(got - h.oracle(rows)).max() < 5e-5


def test_matrix_memory_unequal_sequences_in_one_step():
    h = MemoryHarness(2, 12, 10)
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
def test_matrix_memory_carries_one_early_token_over_hundreds(decoded):
    """Only one token writes along e0 and nothing decays: hundreds of tokens later a query along e0 still reads its value."""
    H, D, Dv, T, star = 2, 16, 12, 330, 4
    h = MemoryHarness(H, D, Dv, cap=30.0)
    h.ib[:], h.fb[:] = 0.0, 60.0                                         # forget gate at log sigmoid(30): everything is kept
    rng = np.random.default_rng(1)
    rows = h.random_rows(T, 5)
    q, k = np.zeros((T, H, D)), 0.3 * rng.standard_normal((T, H, D))
    q[:, :, 0] = 5.0
    k[:, :, 0] = 0.0
    k[star, :, 0] = 4.0
    rows[:, :H * D], rows[:, H * D:2 * H * D] = q.reshape(T, -1), k.reshape(T, -1)
    rows[:, -2 * H:] = 0.0
    ref = h.oracle(rows)
    sizes = [star + 2] + [1] * (T - star - 2) if decoded else [100, 130, 100]
    got = np.concatenate([h.run([(0, rows[a:b])])[0] for a, b in cuts_of(sizes)])
    assert np.abs(got - ref).max() < 5e-5
    v = rows[star, 2 * H * D:2 * H * D + H * Dv].reshape(H, Dv)
    want = (R.unit_rms(v, 1e-6).reshape(-1) * h.w) * R.sigmoid(rows[:, 2 * H * D + H * Dv:2 * H * D + 2 * H * Dv])
    assert np.abs(got[star:] - want[star:]).max() < 1e-3                 # the star's value alone, normalised
    assert np.abs(got[:star]).max() < 1e-6


@pytest.mark.parametrize("i_bias,f_bias", [(-8.0, 8.0), (8.0, -8.0), (-8.0, -8.0), (8.0, 8.0)])
def test_matrix_memory_with_gates_at_their_caps(i_bias, f_bias):
    """Strong and faint gates: the running maximum that starts at 0 (faint inputs stay faint at first), the e^-m floor of the
    denominator, states forgotten within a token, and long sums of log gates."""
    h = MemoryHarness(2, 10, 8, cap=6.0)
    h.ib[:], h.fb[:] = i_bias, f_bias
    rows = h.random_rows(200, 11)
    rows[:, :2 * h.H * h.D] *= 0.2
    ref = h.oracle(rows)
    got = np.concatenate([h.run([(0, rows[a:b])])[0] for a, b in cuts_of([1, 2, 130] + [1] * 40 + [27])])
    assert np.abs(got - ref).max() < 1e-4


class AttentionHarness:
    """pgk_seq_mixer_prep_rot_ex2 + pgk_seq_attention_ex3 on raw rows [q | k | v]."""

    def __init__(self, H, G, D, Dv, window, pool, scale=0.3, page=4, dims=0, base=50.0, splits=1, norm=True, turn=True, dtype="float32"):
        self.H, self.G, self.D, self.Dv, self.window, self.pool, self.scale, self.splits = H, G, D, Dv, window, pool, scale, splits
        self.dims, self.base, self.norm, self.turn = dims, base, norm, turn
        self.cache = PagedKVCache([(G, D, Dv)], dtype, page, 64, 2, pools=[pool])
        self.qt = api.seq_queries_per_tile(H, G)
        rng = np.random.default_rng(H * 31 + D)
        self.qw, self.kw = rng.uniform(0.5, 1.5, D), rng.uniform(0.5, 1.5, D)
        self.inv_freq = f64([base ** (-2.0 * i / dims) for i in range(dims // 2)]) if dims else None
        self.v_freq = f64([base ** (-2.0 * i / Dv) for i in range(Dv // 2)]) if turn else None
        self.tickets = gk.zeros((4096,), gk.int32)
        self.cols = H * D + G * D + G * Dv

    def run(self, seq, q, k, v):
        n = q.shape[0]
        slot, pos0 = self.cache.extend(seq, n)
        self.cache.sync_table()
        c, H, G, D, Dv = self.cache, self.H, self.G, self.D, self.Dv
        proj = f32(np.concatenate([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], axis=1))
        single = 1 if n == 1 and pos0 > 0 else 0
        pk, pv = (c.pk[0].device_ptr, c.pv[0].device_ptr) if self.pool else (None, None)
        vf = self.v_freq.device_ptr if self.turn else None
        api.seq_mixer_prep_rot_ex2(proj.device_ptr, self.cols, n, H, G, D, Dv, 0, H * D, H * D + G * D, self.dims,
                                   self.inv_freq.device_ptr if self.dims else None, 2 if self.norm else 0, f32(self.qw).device_ptr,
                                   f32(self.kw).device_ptr, 1e-6, None, None, None, None, 1, 1, vf, self.pool, c.pool_rows(0), pk, pv,
                                   single, c.k[0].device_ptr, c.v[0].device_ptr, c.dtype_code, c.table_dev.device_ptr,
                                   c.pool.max_pages, c.page_size, i32([slot] * n).device_ptr, i32(np.arange(pos0, pos0 + n)).device_ptr,
                                   None)
        tiles = [(i, min(self.qt, n - i), slot, pos0 + i) for i in range(0, n, self.qt)]
        out = keep(gk.zeros((n, H * Dv), gk.float32))
        api.seq_attention_ex3(proj.device_ptr, self.cols, 0, None, 0, 0, 0, out.device_ptr, H * Dv, c.k[0].device_ptr,
                              c.v[0].device_ptr, D, Dv, c.dtype_code, c.table_dev.device_ptr, c.pool.max_pages, c.page_size,
                              i32(tiles).device_ptr, len(tiles), None, None, None, H, G, D, Dv, 0, self.window, 0, self.scale, 0.0, 0,
                              None, 1.0, self.pool, c.pool_rows(0), pk, pv, vf, 1, self.splits,
                              keep(gk.zeros((n * H * self.splits * (Dv + 2),), gk.float32)).device_ptr, self.tickets.device_ptr, single,
                              None)
        return out.to_numpy().reshape(n, H, Dv)

    def oracle(self, q, k, v):
        p = np.arange(len(q))
        if self.norm:
            q, k = R.unit_rms(q, 1e-6) * self.qw, R.unit_rms(k, 1e-6) * self.kw
        if self.dims:
            q, k = R.rotate_pairs(q, p, self.dims, self.base), R.rotate_pairs(k, p, self.dims, self.base)
        if self.turn:
            v = R.rotate_pairs(v, p, self.Dv, self.base)
        o = R.pooled_window_attention(q, k, v, self.scale, self.window, self.pool)
        return R.rotate_pairs(o, p, self.Dv, self.base, -1.0) if self.turn else o


# block sizes that divide a page, straddle pages, exceed a page, equal 1; windows of 1, below a block, beyond the sequence, none
ATTENTION_LAYOUTS = [dict(H=4, G=2, D=16, Dv=8, window=7, pool=2, dims=8), dict(H=6, G=2, D=8, Dv=12, window=3, pool=4, dims=8, page=3),
                     dict(H=3, G=3, D=12, Dv=20, window=100, pool=4, dims=4), dict(H=2, G=1, D=40, Dv=72, window=20, pool=3, dims=12, page=8),
                     dict(H=1, G=1, D=6, Dv=70, window=1, pool=5, dims=2), dict(H=2, G=2, D=10, Dv=10, window=0, pool=0, dims=10),
                     dict(H=4, G=1, D=8, Dv=130, window=5, pool=1, dims=6, page=2), dict(H=2, G=1, D=4, Dv=34, window=9, pool=11, dims=4, page=4),
                     dict(H=40, G=1, D=8, Dv=6, window=6, pool=3, dims=2, page=16), dict(H=2, G=2, D=9, Dv=7, window=4, pool=3, dims=4, turn=False),
                     dict(H=2, G=1, D=16, Dv=16, window=8, pool=7, dims=16, norm=False, page=64)]


@pytest.mark.parametrize("layout", ATTENTION_LAYOUTS)
def test_pooled_attention_agrees_with_the_oracle(layout):
    h = AttentionHarness(**layout)
    rng = np.random.default_rng(h.H * 7 + h.D)
    T = 75
    q, k, v = rng.standard_normal((T, h.H, h.D)), rng.standard_normal((T, h.G, h.D)), rng.standard_normal((T, h.G, h.Dv))
    ref = h.oracle(q, k, v)
    for name, sizes in (("whole", [T]), ("portions", [2, 2, 9, 1, 17, 14, 30]), ("decoded", [5] + [1] * 70), ("from zero", [1] * 30 + [45])):
        got = np.concatenate([h.run(name, q[a:b], k[a:b], v[a:b]) for a, b in cuts_of(sizes)])
        assert np.abs(got - ref).max() < 3e-5, name
        h.cache.release(name)                                            # the next one inherits its pages and pooled rows


@pytest.mark.parametrize("splits", [2, 3, 7])
@pytest.mark.parametrize("n_last", [1, 6])
def test_pooled_attention_in_key_slices(splits, n_last):
    h = AttentionHarness(4, 2, 12, 14, window=30, pool=4, dims=8, page=8, splits=splits)
    rng = np.random.default_rng(splits)
    T = 400
    q, k, v = rng.standard_normal((T, 4, 12)), rng.standard_normal((T, 2, 12)), rng.standard_normal((T, 2, 14))
    h.run("a", q[:T - n_last], k[:T - n_last], v[:T - n_last])
    got = h.run("a", q[T - n_last:], k[T - n_last:], v[T - n_last:])
    assert np.abs(got - h.oracle(q, k, v)[T - n_last:]).max() < 3e-5


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("window,pool,page", [(9, 4, 4), (64, 8, 16), (65, 5, 64), (6, 7, 4), (130, 16, 64)])
def test_standout_token_in_the_window_in_the_gap_and_in_its_block(window, pool, page, decoded):
    """One key outweighs all others: its token is seen for `window` positions, then by nobody until its block has left the
    window too, then through the block's mean for good."""
    H, G, D, Dv = 2, 1, 8, 4
    for star in (0, pool - 1, pool, page - 1, page, 2 * pool + 1):
        b_end = star // pool * pool + pool - 1
        T = max(star + window + 4, b_end + window + 4)
        rng = np.random.default_rng(star)
        q = np.zeros((T, H, D))
        q[:, :, 4] = 10.0
        k = 0.1 * rng.standard_normal((T, G, D))
        k[:, :, 4] = -1.0
        k[star, 0, 4] = 2.0 * pool + 6.0                                 # the block's mean stands out as well
        v = 0.01 * rng.standard_normal((T, G, Dv))
        v[star, 0, 1] = 2.0 * pool
        h = AttentionHarness(H, G, D, Dv, window, pool, scale=3.0, page=page, dims=4, norm=False, turn=False)
        n0 = star + 1 if decoded else T - 3
        got = np.concatenate([h.run("a", q[:n0], k[:n0], v[:n0])] + [h.run("a", q[i:i + 1], k[i:i + 1], v[i:i + 1]) for i in range(n0, T)])
        assert np.abs(got - h.oracle(q, k, v)).max() < 1e-4
        for i in range(T):
            as_token, as_block = 0 <= i - star < window, b_end <= i - window
            want = 2.0 * pool if as_token else (2.0 if as_block else 0.0)      # never both: the block waits for its last token
            assert np.abs(got[i, :, 1] - want).max() < 0.1, (star, i)


@pytest.mark.parametrize("decoded", [False, True])
def test_far_block_among_hundreds(decoded):
    """The query's score picks one block of ten thousand tokens' worth far back, at page borders and beside them."""
    H, G, D, Dv, window, pool, page, T = 1, 1, 4, 2, 16, 4, 8, 900
    for b in (0, 1, 2, 111, 219):
        q, k, v = np.zeros((T, H, D)), np.zeros((T, G, D)), np.zeros((T, G, Dv))
        q[:, :, 0] = 6.0
        k[b * pool:(b + 1) * pool, :, 0] = 6.0
        v[:, :, 0] = 0.01 * np.arange(T)[:, None]
        h = AttentionHarness(H, G, D, Dv, window, pool, scale=1.0, page=page, norm=False, turn=False)
        n0 = T - 5 if decoded else T
        out = [h.run("a", q[:n0], k[:n0], v[:n0])] + [h.run("a", q[i:i + 1], k[i:i + 1], v[i:i + 1]) for i in range(n0, T)]
        got = np.concatenate(out)[-5:, 0, 0]
        assert np.abs(got - 0.01 * (b * pool + (pool - 1) / 2)).max() < 1e-4, b


def test_norm_in_front_of_the_rotation_and_behind_it_differ_and_are_both_right():
    H, D, dims, base = 1, 8, 8, 30.0
    rng = np.random.default_rng(0)
    q, w = rng.standard_normal((9, H, D)), rng.uniform(0.2, 2.0, D)
    f = f64([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    cache = PagedKVCache([(1, D, 2)], "float32", 4, 16, 1)
    cache.extend("a", 9)
    cache.sync_table()
    p = np.arange(9)
    for pairs in (0, 1):
        for first in (0, 1):
            proj = f32(np.concatenate([q.reshape(9, D), q.reshape(9, D), np.zeros((9, 2))], axis=1))
            api.seq_mixer_prep_rot_ex2(proj.device_ptr, 2 * D + 2, 9, H, 1, D, 2, 0, D, 2 * D, dims, f.device_ptr, 2, f32(w).device_ptr,
                                       f32(w).device_ptr, 1e-6, None, None, None, None, pairs, first, None, 0, 0, None, None, 0,
                                       cache.k[0].device_ptr, cache.v[0].device_ptr, 0, cache.table_dev.device_ptr, cache.pool.max_pages,
                                       4, i32([0] * 9).device_ptr, i32(p).device_ptr, None)
            half = np.concatenate([np.arange(0, D, 2), np.arange(1, D, 2)])       # half layout = pairs under this order

            def rot(x):
                if pairs:
                    return R.rotate_pairs(x, p, dims, base)
                y = np.empty_like(x)
                y[..., half] = x
                y = R.rotate_pairs(y, p, dims, base)
                return y[..., half]
            want = rot(R.unit_rms(q, 1e-6) * w) if first else R.unit_rms(rot(q), 1e-6) * w
            assert np.abs(proj.to_numpy()[:, :D].reshape(9, H, D) - want).max() < 1e-5, (pairs, first)


# ================================================================ whole models
def variants():
    """Sizes that the mechanisms must not assume equal or 1: key and value sizes, head counts, rotated dimensions below the head
    size and equal to it, a window of one, below a block, beyond the sequence and none, blocks of one token, of a page and of no
    divisor of it, one chosen expert and all of them, shared experts narrower, as wide and wider than the others and none,
    layers without feed-forward, odd widths, every order of layers, values wider than one block's columns."""
    yield "base", R.make_config([R.mlstm_layer(mlp=R.dense_ff()), R.attention_layer(mlp=R.moe_ff()), R.mlstm_layer(mlp=R.moe_ff(shared_ff=12))])
    yield "attention_first", R.make_config([R.attention_layer(heads=6, kv_heads=3, dim=10, vdim=4, dims=10, window=5, pool=3, mlp=R.moe_ff(top=1, shared_ff=20)),
                                            R.mlstm_layer(heads=2, dim=5, vdim=9, gate_cap=2.0, mlp=R.dense_ff(31)),
                                            R.attention_layer(heads=2, kv_heads=1, dim=16, vdim=20, dims=2, window=1, pool=1)],
                                           vocab=61, width=52, logit_scale=1.7)
    yield "wide_values", R.make_config([R.mlstm_layer(heads=1, dim=70, vdim=140, mlp=R.moe_ff(experts=3, top=3, ff=8, shared_ff=0)),
                                        R.attention_layer(heads=3, kv_heads=3, dim=6, vdim=6, dims=4, window=2, pool=7, mlp=None),
                                        R.attention_layer(heads=1, kv_heads=1, window=1000, pool=4, mlp=R.dense_ff(7))], width=33, vocab=47)
    yield "only_attention", R.make_config([R.attention_layer(window=0, mlp=R.moe_ff(experts=40, top=35, ff=5, shared_ff=3)),
                                           R.attention_layer(heads=5, kv_heads=5, window=16, pool=16, base=1e4)])
    yield "only_memory", R.make_config([R.mlstm_layer(), R.mlstm_layer(heads=4, dim=8, vdim=8, gate_cap=15.0, mlp=R.dense_ff(16))])


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
    got += [m.step([("a", [t], [0])]) for t in toks[9:]]                 # windows and blocks pass over decoded tokens
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


@pytest.mark.parametrize("name", ["base", "attention_first", "wide_values"])
def test_batch_of_unequal_requests_equals_each_alone(name):
    cfg, P, m = make(name, tokens_hint=16)                               # small pool: pages (with pooled rows) and slots (with state) grow
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


def test_pages_slots_state_and_pooled_rows_are_used_again():
    cfg, P, m = make("base", page=4)
    a, b, c = tokens(cfg, 39, seed=20), tokens(cfg, 14, seed=21), tokens(cfg, 42, seed=22)
    m.step([("a", a, []), ("b", b[:6], [])])
    pages_a, slot_a = m.cache.pool.page_list("a"), m.cache.pool.slot("a")
    m.step([("b", b[6:], [])], end=["a"])
    got = m.step([("c", c[:13], list(range(13)))])                       # c inherits a's slot (dirty state) and pages (with their blocks)
    assert m.cache.pool.slot("c") == slot_a and set(m.cache.pool.page_list("c")) <= set(pages_a)
    got = np.concatenate([got] + [m.step([("c", [t], [0]), ("b", [1], [])])[:1] for t in c[13:]])
    assert np.abs(got - R.forward(cfg, P, c)).max() < F32_TOL
    m.release("c")
    got = np.concatenate([m.step([("d", [t], [0]), ("b", [2], [])])[:1] for t in c[:16]])     # and a sequence decoded from 0 in it
    assert np.abs(got - R.forward(cfg, P, c[:16])).max() < F32_TOL


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
    wrong = [(t + 1) % cfg["vocab"] for t in toks]
    m.step([("a", toks[:33] + wrong[33:], [])])
    m.cache.truncate("a", 33)                                            # blocks over the cut are pooled again
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
    cfg = layered_config_from_json(R.make_config([R.attention_layer(heads=4, kv_heads=2, dim=32, vdim=32, dims=16, window=20, pool=8, mlp=R.dense_ff(128)),
                                                  R.mlstm_layer(heads=4, dim=32, vdim=64, mlp=R.moe_ff(experts=4, top=2, ff=64, shared_ff=96)),
                                                  R.mlstm_layer(heads=2, dim=32, vdim=160, mlp=R.moe_ff(experts=4, top=2, ff=64, shared_ff=64))],
                                                 vocab=256, width=128))
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
    assert isinstance(m, llm.LayeredCausalModel) and m.config.architecture == "Vosolorn"
    toks = tokens(cfg, 30)
    assert np.abs(m.step([("a", toks, list(range(30)))]) - R.forward(cfg, P, toks)).max() < F32_TOL
    with pytest.raises(ValueError, match="shape"):
        bad = dict(P)
        bad["l0.mix.q.norm"] = P["l0.mix.q.norm"][:-1]
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
