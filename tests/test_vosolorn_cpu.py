"""CPU tests of the Vosolorn design: config parsing and registry (every size different, rejections), the state and the pooled
rows the cache manager is asked for, and the oracle's own mechanisms on hand-made cases whose answer is known."""
import numpy as np
import pytest

from pygpukit_b200.llm.config import AttentionMixerSpec, MatrixLSTMSpec, LAYERED_ARCHITECTURES, MoESpec, layered_config_from_json
from tests import vosolorn_ref as R


def test_config_reads_every_size_and_constant_from_the_file():
    cfg = R.make_config([R.attention_layer(heads=6, kv_heads=3, dim=10, vdim=14, dims=6, base=777.0, scale=0.21, window=13, pool=5,
                                           mlp=R.dense_ff(50)),
                         R.mlstm_layer(heads=5, dim=12, vdim=7, gate_cap=3.5, mlp=R.moe_ff(experts=7, top=4, ff=21, shared_ff=33)),
                         R.mlstm_layer(heads=2, dim=4, vdim=9, gate_cap=30.0, mlp=R.moe_ff(experts=3, top=1, ff=9, shared_ff=5)),
                         R.mlstm_layer(mlp=R.moe_ff(shared_ff=0)), R.mlstm_layer()],
                        vocab=77, width=44, eps=3e-6, logit_scale=0.125)
    c = layered_config_from_json(cfg)
    assert "vosolorn" in LAYERED_ARCHITECTURES and c.architecture == "Vosolorn"
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.logit_scale) == (77, 44, 3e-6, 0.125)
    assert (c.block, c.norm, c.tied_head, c.embed_norm, c.layer_scale) == ("post_norm", "rmsnorm", True, True, True)
    a, m, m2 = (L.mixer for L in c.layers[:3])
    assert isinstance(a, AttentionMixerSpec) and (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.pool) == (6, 3, 10, 14, 0.21, 13, 5)
    assert (a.rot.dims, a.rot.base, a.rot.factor, a.rot.layout) == (6, 777.0, 1.0, "pairs")
    assert a.rot.value_inv_freq(14) == [777.0 ** (-2.0 * i / 14) for i in range(7)]
    assert a.qk_norm and a.norm_weight and a.norm_first and a.rot_values and not a.out_gate and a.weights == "softmax"
    assert a.sink == "none" and a.keep_first == 0 and a.chunk == 0 and a.slopes() == []
    assert a.proj_cols == 6 * 10 + 3 * 10 + 3 * 14 and a.cache_shape() == (3, 10, 14) and a.state_shapes == ()
    assert isinstance(m, MatrixLSTMSpec) and (m.heads, m.dim, m.vdim, m.gate_cap) == (5, 12, 7, 3.5)
    assert m.proj_cols == 2 * 5 * 12 + 2 * 5 * 7 + 10 and m.attn_cols == 35 and m.cache_shape() == (0, 0, 0)
    assert m.state_shapes == (5 * 12 * 7, 5 * 12, 5) and m2.state_shapes == (2 * 4 * 9, 8, 2)
    f0, f1, f2, f3, f4 = (L.mlp for L in c.layers)
    assert (f0.kind, f0.ff, f0.activation) == ("dense", 50, "gelu_tanh") and f4 is None
    assert (f1.experts, f1.top, f1.ff, f1.shared_ff, f1.router, f1.activation) == (7, 4, 21, 33, "logits", "gelu")
    assert not f1.shared_slot and f1.slots == 4                          # wider than the experts: products of its own
    assert f2.shared_slot and f2.slots == 2 and not f3.shared_slot and f3.slots == 3
    assert not MoESpec(4, 2, 8, shared_ff=8).shared_slot                 # only behind the router it was built for


def test_config_without_a_window_sees_every_token_and_pools_nothing():
    cfg = R.make_config([R.attention_layer()])
    del cfg["layers"][0]["mixer"]["mask"]
    a = layered_config_from_json(cfg).layers[0].mixer
    assert a.window == 0 and a.pool == 0


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "key/value heads"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=7), "turn in pairs"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rotated dimensions"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "without a rotation"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(pool=-1), "blocks of -1"),
    (lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0), "gate cap"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "feed-forward kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top 9"),
])
def test_config_rejections(change, match):
    cfg = R.make_config([R.attention_layer(), R.mlstm_layer(mlp=R.moe_ff())])
    change(cfg)
    with pytest.raises(ValueError, match=match):
        layered_config_from_json(cfg)


def test_oracle_rotation_in_pairs():
    x = np.zeros((2, 1, 6))
    x[:, 0] = [1, 0, 0, 1, 5, 7]
    y = R.rotate_pairs(x, [0, 3], 4, 100.0)
    assert np.allclose(y[0], x[0])
    c1, s1 = np.cos(3 * 100.0 ** -0.5), np.sin(3 * 100.0 ** -0.5)        # second pair: base^(-2/4)
    assert np.allclose(y[1, 0], [np.cos(3.0), np.sin(3.0), -s1, c1, 5, 7])
    assert np.allclose(R.rotate_pairs(y, [0, 3], 4, 100.0, -1.0), x)     # turning back undoes it


def test_oracle_rotated_values_turned_back_depend_on_the_distance_alone():
    rng = np.random.default_rng(0)
    v = rng.standard_normal((1, 1, 8))
    far = R.rotate_pairs(R.rotate_pairs(v, [40], 8, 50.0), [47], 8, 50.0, -1.0)
    near = R.rotate_pairs(R.rotate_pairs(v, [3], 8, 50.0), [10], 8, 50.0, -1.0)
    assert np.allclose(far, near) and not np.allclose(far, v)


@pytest.mark.parametrize("window,pool,i,tokens,blocks", [
    (5, 3, 2, [0, 1, 2], []),
    (5, 3, 6, [2, 3, 4, 5, 6], []),                                      # 0 and 1 have left, their block (0 .. 2) has not
    (5, 3, 7, [3, 4, 5, 6, 7], [0]),                                     # 2 = 7 - 5: the block is seen
    (5, 3, 9, [5, 6, 7, 8, 9], [0]),
    (5, 3, 10, [6, 7, 8, 9, 10], [0, 1]),
    (1, 1, 3, [3], [0, 1, 2]),
    (2, 4, 5, [4, 5], [0]),
    (4, 0, 6, [3, 4, 5, 6], []),
    (0, 3, 2, [0, 1, 2], []),
])
def test_oracle_visible_tokens_and_blocks(window, pool, i, tokens, blocks):
    assert R.window_and_blocks(i, window, pool) == (tokens, blocks)


def test_oracle_pooled_attention_in_closed_form():
    T, window, pool = 9, 2, 3
    q, k = np.zeros((T, 1, 2)), np.zeros((T, 1, 2))                      # every score 0: a plain mean over what is seen
    v = np.arange(float(T)).reshape(T, 1, 1)
    o = R.pooled_window_attention(q, k, v, 1.0, window, pool)[:, 0, 0]
    want = [0, 0.5, 1.5, 2.5, (1 + 3 + 4) / 3, (1 + 4 + 5) / 3, (1 + 5 + 6) / 3, (1 + 4 + 6 + 7) / 4, (1 + 4 + 7 + 8) / 4]
    assert np.allclose(o, want)


def test_oracle_matrix_memory_in_closed_form():
    T = 4
    q, k = np.ones((T, 1, 1)), np.ones((T, 1, 1))
    v = np.arange(1.0, T + 1).reshape(T, 1, 1)
    i, f = np.zeros((T, 1)), np.full((T, 1), np.log(0.5))
    # unscaled: S_t = S/2 + v, n_t = n/2 + 1, denominator max(|n|, 1) with the running maximum at 0 (i = 0 wins)
    o = R.mlstm_recurrence(q, k, v, i, f)[:, 0, 0]
    S = n = 0.0
    for t in range(T):
        S, n = 0.5 * S + (t + 1), 0.5 * n + 1.0
        assert np.isclose(o[t], S / (max(n, 1.0) + 1e-6))
    # the maximum starts at 0, not at minus infinity: with f = 0 it stays there, and a faint input stays faint against e^-m = 1
    o = R.mlstm_recurrence(q, k, v, np.full((T, 1), -5.0), np.zeros((T, 1)))[:, 0, 0]
    assert np.allclose(o, np.exp(-5.0) * np.array([1, 3, 6, 10]) / (1.0 + 1e-6))


def test_oracle_router_weighs_the_chosen_alone():
    z = np.array([[0.0, 3.0, -1.0, 2.0]])
    order, w = R.route(z, 2)
    assert order.tolist() == [[1, 3]] and np.allclose(w, [[1 / (1 + np.exp(-1.0)), 1 / (1 + np.exp(1.0))]])


def test_oracle_the_two_forms_of_gelu():
    z = np.array([-3.0, -0.5, 0.0, 1.0, 4.0])
    assert np.allclose(R.gelu_erf(z), [-3 * 0.001349898, -0.15426877, 0, 0.84134475, 3.99987331])
    d = np.abs(R.gelu_erf(z) - R.gelu_tanh(z))
    assert d.max() < 1e-3 and d.max() > 1e-5                             # alike, and not the same
