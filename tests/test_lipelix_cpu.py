"""The Lipelix design, host side: registry, and the oracle's own invariants."""
import copy

import numpy as np
import pytest

import decoder_cases as dc
import lipelix_cases as lc
from jgpt_b200 import decoder as D
from jgpt_b200 import registry
from oracle import lipelix_ref as L


def test_registry_reads_every_size_and_constant():
    cfg = lc.config([lc.gen(heads=5, dim=11, mlp=lc.dense(20)), lc.win(heads=6, kv_heads=3, dim=10, vdim=18, rot_dims=8, base=70.0, scale=0.31, size=9, keep=4),
                     lc.att(heads=9, kv_heads=3, dim=12, vdim=18, rot_dims=4, mlp=lc.dense(28)), lc.att(v_mix=False, mlp=None)], mult=0.45, scale=3.5)
    W = lc.weights(cfg, rank=7)
    d = registry.describe(cfg, lambda n: W[n].shape)
    assert (d.vocab, d.width, d.eps, d.embed_scale, d.residual_mult, d.norm, d.norm_both, d.token_shift, d.residual_gate, d.head, d.pos_table) == (
        101, 72, 3e-6, 3.5, 0.45, D.NORM_RMS, True, True, True, True, False)
    g, w, a, b = (x.branches[0] for x in d.layers)
    assert [x.ff for x in d.layers] == [20, 44, 28, 0] and {x.ff_kind for x in d.layers} == {D.FF_RELU2}
    assert (g.kind, g.heads, g.kv_heads, g.dim, g.vdim, g.rank_a) == (D.MIX_GENERAL_DELTA, 5, 5, 11, 11, 7) and np.isclose(g.decay_rate, np.exp(-0.5))
    assert (w.kind, w.heads, w.kv_heads, w.dim, w.vdim, w.window, w.keep, w.sink, w.qk_norm, w.v_mix, w.chunk) == (
        D.MIX_ATTENTION, 6, 3, 10, 18, 9, 4, D.SINK_ZERO, D.QK_NORM_UNIT, True, 0)
    assert (w.rot_dims, w.rot_base, w.rot_interleaved, w.rot_factor, w.score_scale) == (8, 70.0, False, 0, 0.31)
    assert (a.heads, a.kv_heads, a.window, a.keep, a.sink, a.qk_norm, a.v_mix, a.rot_dims) == (9, 3, 0, 0, D.SINK_LEARNED, D.QK_NORM_ALL, True, 4)
    assert (b.v_mix, b.qkv_bias, b.gate, b.maps) == (False, False, D.GATE_NONE, 1)
    # nothing is left over but the share of the layer that the values come from, nothing is made up
    assert {n for *_, n in d.all_tensors()} == set(W) - {"l1.mix.vmix"}


def test_unknown_parts_are_refused():
    cfg = lc.config([lc.att()])
    shape = lambda n: lc.weights(cfg)[n].shape  # noqa: E731
    for key, value, what in (("type", "mystery", "mixer type"), ("mlp", {"kind": "sparse", "ff": 4}, "feed-forward")):
        bad = copy.deepcopy(cfg)
        bad["layers"][0][key] = value
        with pytest.raises(ValueError, match=what):
            registry.describe(bad, shape)


def test_window_and_kept_tokens():
    ok = L.visible(12, {"size": 3, "keep_first": 2})
    for i in range(12):
        assert [j for j in range(12) if ok[i, j]] == sorted({j for j in range(12) if j <= i and (i - j < 3 or j < 2)})
    assert ok[11].sum() == 5 and ok[0].sum() == 1 and L.visible(12)[11].sum() == 12


def test_sinks_take_their_share():
    s = np.array([[1.0, 2.0, -np.inf]])
    p = L.sink_softmax(s, 0.0)
    assert np.allclose(p, np.exp(s) / (1 + np.exp(1) + np.exp(2)))
    assert np.allclose(L.sink_softmax(s, -1e9).sum(), 1) and L.sink_softmax(s, 60.0).sum() < 1e-20


def test_unit_norm_and_rotation_commute():
    x = np.random.default_rng(0).standard_normal((7, 2, 10))
    rot = {"base": 40.0, "dims": 6}
    unit = lambda y: L.rms_norm(y, 1.0, 1e-5)  # noqa: E731
    assert np.allclose(unit(L.rotate(x, rot)), L.rotate(unit(x), rot)) and np.allclose(L.rotate(x, rot)[..., 6:], x[..., 6:])


def test_general_delta_scan_by_hand():
    """Without removal a plain sum that decays; with full removal and no decay a key's old value is taken out before the new one."""
    k = np.zeros((3, 1, 4))
    k[0, 0, 1], k[1, 0, 2], k[2, 0, 1] = 2.0, 1.0, 2.0
    v, r, one = np.arange(9.0).reshape(3, 1, 3) + 1, np.tile([0.0, 1.0, 10.0, 0.0], (3, 1, 1)), np.ones((3, 1, 4))
    plain = L.general_delta_scan(r, k, v, 0.5 * one, 0 * one)
    assert np.allclose(plain[2, 0], 2 * (0.25 * v[0, 0] + v[2, 0]) + 10 * 0.5 * v[1, 0])
    removed = L.general_delta_scan(r, k, v, one, one)
    assert np.allclose(removed[2, 0], 2 * v[2, 0] + 10 * v[1, 0], atol=1e-5)


def test_values_come_from_the_first_mixing_layer():
    cfg = lc.config([lc.att(v_mix=False), lc.win(), lc.att(vdim=6, kv_heads=4, heads=8)])
    W, t = lc.weights(cfg), np.arange(1, 9)
    base = L.forward(cfg, W, t)
    assert np.allclose(base, L.forward(cfg, {**W, "l1.mix.vmix": np.array(0.1)}, t))  # the source's own share is not read
    full = L.forward(cfg, {**W, "l2.mix.vmix": np.array(1.0)}, t)
    assert not np.allclose(base, full) and np.allclose(full, L.forward(cfg, {**W, "l2.mix.vmix": np.array(1.0), "l2.mix.v": 0 * W["l2.mix.v"]}, t))


def test_shift_reads_the_row_before():
    h = np.random.default_rng(1).standard_normal((5, 6))
    s = L.shifted(h, np.array([0, 1, 0.5, 0, 1, 2.0]))
    assert np.allclose(s[:, 0], h[:, 0]) and np.allclose(s[1:, 1], h[:-1, 1]) and s[0, 1] == 0 and np.allclose(s[3, 5], 2 * h[2, 5] - h[3, 5])


def test_oracle_is_causal():
    cfg = lc.config([lc.att(), lc.gen(), lc.win(mlp=None), lc.att(mlp=None)])
    W = lc.weights(cfg)
    a = dc.tokens(cfg, 24)
    b = a.copy()
    b[15] = b[15] % (cfg["vocab"] - 1) + 1
    x, y = L.forward(cfg, W, a), L.forward(cfg, W, b)
    assert np.allclose(x[:15], y[:15]) and all(not np.allclose(x[i], y[i]) for i in (15, 16, 23))
