"""CPU tests of the Goluzen design: config parsing and registry (every size different, rejections), what the cache manager is asked
for, and the oracle's own mechanisms on hand-made cases whose answer is known."""
import math

import numpy as np
import pytest

from pygpukit_b200.llm.config import (LAYERED_ARCHITECTURES, AttentionMixerSpec, GLAMixerSpec, LatentMixerSpec, MoESpec, YarnSpec,
                                      layered_config_from_json)
from tests import goluzen_ref as R


def test_config_reads_every_size_and_constant_from_the_file():
    cfg = R.make_config([R.latent_layer(heads=5, dim=9, rot_dim=6, vdim=7, kv_rank=13, scale=0.31, window=17, base=777.0, factor=3.0,
                                        original=80, fast=5.0, slow=2.0, mlp=R.dense_ff(50)),
                         R.gla_layer(heads=4, dim=12, vdim=11, tau=3.5, mlp=R.moe_ff(experts=8, top=3, ff=21, shared_ff=33, groups=(4, 2), scale=0.4)),
                         R.attention_layer(heads=6, kv_heads=3, dim=10, vdim=14, dims=4, base=55.0, factor=2.5, scale=0.21, softcap=9.0,
                                           window=19, keep_first=2, mlp=R.moe_ff(experts=3, top=1, ff=9, shared_ff=5, groups=None)),
                         R.latent_layer(heads=2, dim=4, rot_dim=6, vdim=3, kv_rank=13, scale=0.9, window=5, base=777.0, factor=3.0,
                                        original=80, fast=5.0, slow=2.0, kv_from=0), R.gla_layer(mlp=R.moe_ff(shared_ff=0))],
                        vocab=77, width=44, eps=3e-6, embed_scale=2.25)
    c = layered_config_from_json(cfg)
    assert "goluzen" in LAYERED_ARCHITECTURES and c.architecture == "Goluzen"
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.embed_scale) == (77, 44, 3e-6, 2.25)
    assert (c.block, c.norm, c.tied_head, c.embed_norm) == ("pre_norm", "rmsnorm_1p", False, False)
    a, g, t, b, _ = (L.mixer for L in c.layers)
    assert isinstance(a, LatentMixerSpec) and (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.scale, a.window) == (5, 9, 6, 7, 13, 0.31, 17)
    assert (a.q_rank, a.rot_dims, a.rot_base, a.yarn, a.kv_from, a.sink) == (0, 6, 777.0, YarnSpec(3.0, 80.0, 5.0, 2.0), -1, "none")
    assert a.out_gate and not a.gate_per_head and a.proj_cols == 5 * 15 + 19 + 35 and a.cache_shape() == (1, 19, 0)
    assert b.kv_from == 0 and b.proj_cols == 2 * 10 + 6 and b.cache_shape() == (0, 0, 0) and b.window == 5
    assert isinstance(g, GLAMixerSpec) and (g.heads, g.dim, g.vdim, g.tau, g.gate_rank) == (4, 12, 11, 3.5, 0)
    assert g.state_shapes == (4 * 12 * 11,) and g.cache_shape() == (0, 0, 0) and g.attn_cols == 44 and g.proj_cols == 2 * 48 + 2 * 44
    assert isinstance(t, AttentionMixerSpec) and (t.heads, t.kv_heads, t.dim, t.vdim, t.scale, t.softcap) == (6, 3, 10, 14, 0.21, 9.0)
    assert (t.window, t.keep_first, t.rot.dims, t.rot.base, t.rot.factor, t.rot.layout) == (19, 2, 4, 55.0, 2.5, "half")
    assert t.qk_norm and not t.norm_weight and not t.norm_first and t.qkv_bias and t.sink == "learned" and not t.out_gate
    f0, f1, f2, f3, f4 = (L.mlp for L in c.layers)
    assert (f0.kind, f0.ff, f0.activation) == ("dense", 50, "gelu_tanh_up") and f3 is None
    assert (f1.experts, f1.top, f1.ff, f1.shared_ff, f1.router, f1.activation) == (8, 3, 21, 33, "sigmoid", "relu2")
    assert (f1.group_count, f1.group_keep, f1.weight_scale, f1.renorm, f1.shared_gate) == (4, 2, 0.4, False, True)
    assert not f1.shared_slot and f1.slots == 3                          # wider than the experts: products of its own
    assert f2.shared_slot and f2.slots == 2 and (f2.group_count, f2.group_keep) == (1, 1)
    assert not f4.shared_slot and not f4.shared_gate
    assert not MoESpec(4, 2, 8, shared_ff=8).shared_slot


def test_config_without_masks_or_position_scaling():
    cfg = R.make_config([R.attention_layer(), R.latent_layer()])
    for L in cfg["layers"]:
        del L["mixer"]["mask"]
        del L["mixer"]["rot"]["scaling"]
    a, b = (L.mixer for L in layered_config_from_json(cfg).layers)
    assert a.window == 0 and a.keep_first == 0 and a.rot.factor == 1.0
    assert b.window == 0 and b.yarn is None and b.rot_mult == 1.0 and b.inv_freq() == [400.0 ** (-2.0 * i / 8) for i in range(4)]


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "key/value heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rotated dimensions"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=-2), "window -2"),
    (lambda c: c["layers"][1]["mixer"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "feed-forward kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top 5"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "4 groups"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10), "rotated dimensions"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "no latent of its own"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=4), "no latent of its own"),
    (lambda c: c["layers"][3]["mixer"].update(kv_rank=15), "differ from layer 2"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(base=401.0), "differ from layer 2"),
])
def test_config_rejections(change, match):
    cfg = R.make_config([R.attention_layer(), R.gla_layer(mlp=R.moe_ff()), R.latent_layer(), R.latent_layer(kv_from=2)])
    change(cfg)
    with pytest.raises(ValueError, match=match):
        layered_config_from_json(cfg)


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [(16, 5e5, 4.0, 1024, 32.0, 1.0), (64, 1e4, 40.0, 4096, 32.0, 1.0), (8, 300.0, 2.0, 30, 1e9, 1e-9),
                                                                 (6, 50.0, 7.0, 10, 1.0, 1.0), (2, 1e4, 1.0, 100, 8.0, 2.0)])
def test_scaled_frequencies_of_the_package_and_of_the_oracle_agree(dims, base, factor, original, fast, slow):
    want, mult = R.stretched_frequencies({"dims": dims, "base": base, "scaling": dict(factor=factor, original=original, fast=fast, slow=slow)})
    y = YarnSpec(factor, float(original), fast, slow)
    assert np.allclose(y.inv_freq(dims, base), want, rtol=1e-14, atol=0) and y.mult == mult
    f = base ** (-2.0 * np.arange(dims // 2) / dims)
    assert (want <= f * (1 + 1e-12)).all() and (want >= f / factor * (1 - 1e-12)).all()
    turns = original * f / (2 * math.pi)
    if fast / slow > 4:                                                  # well outside the ramp: untouched, or fully divided
        assert np.allclose(want[turns > 8 * fast], f[turns > 8 * fast]) and np.allclose(want[turns < slow / 1e3], f[turns < slow / 1e3] / factor)


def test_oracle_rotation_layouts_and_factor():
    x = np.arange(1.0, 7.0).reshape(1, 1, 6)
    half = R.rotate(x, [1], np.array([math.pi / 2]), False)
    assert np.allclose(half[0, 0], [-2, 1, 3, 4, 5, 6])
    half = R.rotate(x, [1], np.array([math.pi / 2, math.pi]), False, 2.0)
    assert np.allclose(half[0, 0], [-6, -4, 2, -8, 5, 6])
    pairs = R.rotate(x, [2], np.array([math.pi / 4, math.pi / 2]), True)
    assert np.allclose(pairs[0, 0], [-2, 1, -3, -4, 5, 6])


def test_oracle_window_with_kept_first_tokens():
    assert R.seen(9, 3, 2) == [0, 1, 7, 8, 9] and R.seen(3, 3, 2) == [0, 1, 2, 3] and R.seen(1, 3, 2) == [0, 1]
    assert R.seen(4, 1, 0) == [4] and R.seen(4, 0, 0) == [0, 1, 2, 3, 4]


def test_oracle_sink_is_counted_once_and_neither_scaled_nor_capped():
    q = k = np.zeros((2, 1, 4))
    v = np.ones((2, 1, 1))
    o = R.softmax_attention(q, k, v, 3.0, softcap=0.5, sinks=np.array([math.log(6.0)]))
    assert np.allclose(o[:, 0, 0], [1 / 7, 2 / 8])


def test_oracle_recurrence_decays_the_key_channels():
    a = np.array([[[0.5, 1.0]]] * 3)
    k, q = np.array([[[1.0, 1.0]], [[0, 0]], [[0, 0]]]), np.array([[[1.0, 0.0]], [[1.0, 0.0]], [[0.0, 1.0]]])
    v = np.array([[[2.0]], [[5.0]], [[7.0]]])
    assert np.allclose(R.decayed_recurrence(q, k, v, a)[:, 0, 0], [2.0, 1.0, 2.0])     # the decay acts before the write


def test_oracle_router_ranks_groups_by_their_two_best_and_weighs_without_the_correction():
    s = np.array([0.9, 0.1, 0.6, 0.55, 0.2, 0.2])
    z = np.log(s / (1 - s))[None]
    zero = np.zeros(6)
    assert R.route(z, zero, 2, 3, 1, 1.0)[0].tolist() == [[2, 3]]        # 0.6 + 0.55 beats 0.9 + 0.1
    chosen, w = R.route(z, zero, 2, 3, 2, 2.0)
    assert chosen.tolist() == [[0, 2]] and np.allclose(w, [[1.8, 1.2]])
    lift = np.array([0, 0, -5.0, -5.0, -5.0, -4.0])                      # every other choice is negative: still only group 0 competes
    chosen, w = R.route(z, lift, 2, 3, 1, 1.0)
    assert chosen.tolist() == [[0, 1]] and np.allclose(w, [[0.9, 0.1]])


def test_oracle_layers_share_a_latent():
    cfg = R.make_config([R.latent_layer(), R.latent_layer(heads=2, window=4, kv_from=0)])
    P = R.random_params(cfg, seed=4)
    assert "l1.mix.dkv" not in P and "l1.mix.dkv.norm" not in P
    toks = [1, 2, 3, 4, 5, 6]
    before = R.forward(cfg, P, toks, True)[1]
    P["l0.mix.uv"] = 2 * P["l0.mix.uv"]                                  # layer 0's own values, not the latent layer 1 reads
    P["l0.mix.o"] = P["l0.mix.o"] / 2
    assert np.allclose(R.forward(cfg, P, toks, True)[1], before)
    P["l0.mix.dkv.norm"] = 2 * P["l0.mix.dkv.norm"]
    P["l0.mix.uk"], P["l0.mix.uv"] = P["l0.mix.uk"] / 2, P["l0.mix.uv"] / 2
    after = R.forward(cfg, P, toks, True)[1]
    assert np.allclose(after[0], before[0]) and np.abs(after[1] - before[1]).max() > 1e-3
