"""The Nefipel design, host side: registry, and the oracle's own invariants."""
import copy

import numpy as np
import pytest

import decoder_cases as dc
import nefipel_cases as nc
from jgpt_b200 import decoder as D
from jgpt_b200 import registry
from oracle import nefipel_ref as N


def test_registry_reads_every_size_and_constant():
    cfg = nc.config([nc.diff(heads=6, kv_heads=3, dim=10, vdim=18, rot_dims=8, base=70.0, scale=0.31, at=0.7, mlp=nc.dense(20)),
                     nc.att(heads=5, kv_heads=1, dim=12, vdim=16, rot_dims=4, mlp=nc.moe(9, 3, 4, 3, 2, ff=24, shared=40)), nc.att(mlp=None),
                     nc.diff(yarn=None, mlp=nc.moe(4, 0, 2, 1, 1, shared=0))], alpha=1.7, scale=3.5)
    W = nc.weights(cfg)
    d = registry.describe(cfg, lambda n: W[n].shape)
    assert (d.vocab, d.width, d.eps, d.embed_scale, d.residual_scale, d.norm, d.norm_after, d.head, d.pos_table) == (
        101, 72, 3e-6, 3.5, 1.7, D.NORM_RMS, True, False, False)
    a, b, c, e = (x.branches[0] for x in d.layers)
    assert [x.ff_kind for x in d.layers] == [D.FF_GATED_RELU, D.FF_MOE, D.FF_GATED_RELU, D.FF_MOE] and [x.ff for x in d.layers] == [20, 24, 0, 28]
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.maps, a.diff, a.gate, a.qkv_bias, a.qk_norm) == (D.MIX_ATTENTION, 6, 3, 10, 18, 2, 0.7, 0, False, True)
    assert (a.rot_dims, a.rot_base, a.rot_interleaved, a.rot_factor, a.rot_original, a.rot_fast, a.rot_slow, a.score_scale) == (8, 70.0, True, 3.0, 60, 8.0, 1.0, 0.31)
    assert (b.heads, b.kv_heads, b.maps, b.gate, b.qkv_bias, b.qk_norm, b.rot_dims, b.rot_interleaved, b.rot_factor) == (5, 1, 1, D.GATE_ELEMENT, True, True, 4, False, 0)
    assert e.rot_factor == 0
    m = d.layers[1].moe
    assert (m.experts, m.identity, m.top, m.groups, m.keep, m.ff, m.shared_ff, m.act, m.shared_act) == (9, 3, 4, 3, 2, 24, 40, D.ACT_RELU2, D.ACT_RELU2)
    assert d.layers[3].moe.shared_ff == 0 and d.layers[0].moe is None
    assert {n for *_, n in d.all_tensors()} == set(W)  # nothing is left over, nothing is made up


def test_unknown_parts_are_refused():
    cfg = nc.config([nc.att()])
    shape = lambda n: nc.weights(cfg)[n].shape  # noqa: E731
    for key, value, what in (("type", "mystery", "mixer type"), ("mlp", {"kind": "sparse", "ff": 4}, "feed-forward")):
        bad = copy.deepcopy(cfg)
        bad["layers"][0][key] = value
        with pytest.raises(ValueError, match=what):
            registry.describe(bad, shape)


@pytest.mark.parametrize("layout", ["half", "interleaved"])
def test_rotation_turns_its_pairs_and_keeps_relative_positions(layout):
    rot = {"base": 50.0, "dims": 6}
    x = np.random.default_rng(0).standard_normal((4, 2, 9))
    y = N.rotate(x, rot, layout)
    assert np.allclose(y[0], x[0]) and np.allclose(y[..., 6:], x[..., 6:])
    pairs = [(0, 3), (1, 4), (2, 5)] if layout == "half" else [(0, 1), (2, 3), (4, 5)]
    for i, (u, v) in enumerate(pairs):
        a = 3 * 50.0 ** (-i / 3)
        assert np.allclose(y[3, :, u], x[3, :, u] * np.cos(a) - x[3, :, v] * np.sin(a)) and np.allclose(y[3, :, v], x[3, :, v] * np.cos(a) + x[3, :, u] * np.sin(a))
    q, k = (N.rotate(np.tile(x[0, i], (9, 1)), rot, layout) for i in range(2))
    s = q @ k.T
    assert np.allclose(np.diag(s, -2), s[2, 0]) and not np.isclose(s[2, 0], s[3, 0])


def test_scaling_slows_only_slow_pairs():
    plain, one = N.frequencies({"base": 1e4, "dims": 32})
    f, mag = N.frequencies({"base": 1e4, "dims": 32, "scaling": {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0}})
    r = plain / f
    assert one == 1 and np.isclose(r[0], 1) and np.isclose(r[-1], 8) and (np.diff(r) > -1e-12).all() and np.isclose(mag, 0.1 * np.log(8) + 1)


def test_choice_scores_may_be_negative_and_weights_ignore_the_correction():
    z = np.log(np.array([0.1, 0.2, 0.3, 0.05, 0.15, 0.2]))
    r = {"top": 2, "groups": {"count": 3, "keep": 2}}
    corr = np.array([-5.0, -5.0, -1.0, -1.2, -2.0, -3.0])  # groups score -4.8, -0.7, -1.85
    got = N.route(z, corr, r)
    assert [e for e, _ in got] == [2, 3] and np.allclose([w for _, w in got], [0.3 / 0.35, 0.05 / 0.35])
    corr[3] = -9.0  # the second group's other member falls behind the third group
    assert [e for e, _ in N.route(z, corr, r)] == [2, 4]
    assert [e for e, _ in N.route(z, corr, {"top": 3, "groups": {"count": 3, "keep": 1}, "identity": 2})][:2] == [2, 3]  # never another group's
    assert np.isclose(N.route_margin(z, corr, r), min(-1.85 + 2.8, -1.85 + 4.8))


def test_differential_maps_cancel():
    rng = np.random.default_rng(1)
    m = nc.diff(heads=2, kv_heads=1, dim=4, vdim=6, at=0.25)["mixer"]
    W = {k[7:]: v for k, v in nc.weights(nc.config([nc.diff(heads=2, kv_heads=1, dim=4, vdim=6)]), 3).items() if k.startswith("l0.mix.")}
    W = {k: np.asarray(v, np.float64) for k, v in W.items()}
    W["o"] = np.eye(12)
    h = rng.standard_normal((5, 72))
    o = N.differential_attention(h, W, m, 1e-9)
    assert np.allclose(np.sqrt((o.reshape(5, 2, 6) ** 2).mean(-1)), 0.75)  # unit size times 1 - diff, whatever the maps
    same = dict(W, lq1=np.zeros(4), lq2=np.zeros(4))
    assert np.isclose(N.difference_factor(same, 0.25), 0.25)


def test_oracle_is_causal():
    cfg = nc.config([nc.att(), nc.diff(), nc.diff(mlp=None), nc.att(mlp=nc.moe())])
    W = nc.weights(cfg)
    a = dc.tokens(cfg, 24)
    b = a.copy()
    b[15] = b[15] % (cfg["vocab"] - 1) + 1
    x, y = N.forward(cfg, W, a), N.forward(cfg, W, b)
    assert np.allclose(x[:15], y[:15]) and all(not np.allclose(x[i], y[i]) for i in (15, 16, 23))
