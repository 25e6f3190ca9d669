"""The Zusepel design, host side: registry, and the oracle's own invariants."""
import copy

import numpy as np
import pytest

import decoder_cases as dc
import zusepel_cases as zc
from jgpt_b200 import decoder as D
from jgpt_b200 import registry
from oracle import zusepel_ref as Z


def test_registry_reads_every_size_and_constant():
    cfg = zc.config([zc.hgrn2(heads=5, dim=12, vdim=20, ff=0), zc.latent(size=33, scale=0.21), zc.wkv(heads=2, dim=16),
                     zc.latent(heads=7, vdim=12, size=9, kv_from=1, ff=36)], mult=0.55)
    W = zc.weights(cfg, rank=6)
    d = registry.describe(cfg, lambda n: W[n].shape)
    assert (d.vocab, d.width, d.eps, d.residual_mult, d.norm, d.head, d.layer_scale, d.depth_average) == (101, 72, 3e-6, 0.55, D.NORM_RMS, True, True, True)
    h, a, w, b = (x.branches[0] for x in d.layers)
    assert [x.ff for x in d.layers] == [0, 52, 44, 36] and all(x.ff_kind == D.FF_XIELU for x in d.layers)
    assert (h.kind, h.heads, h.dim, h.vdim) == (D.MIX_HGRN2, 5, 12, 20)
    assert (w.kind, w.heads, w.dim, w.vdim, w.rank_a) == (D.MIX_WKV, 2, 16, 16, 6)
    assert (a.kind, a.window, a.score_scale, a.q_rank, a.kv_rank, a.rot_dim, a.rot_dims, a.kv_from) == (D.MIX_LATENT, 33, 0.21, 36, 44, 12, 12, 0)
    assert (a.rot_base, a.rot_factor, a.rot_original, a.rot_fast, a.rot_slow) == (300.0, 3.0, 64, 8.0, 1.0)
    assert (b.heads, b.vdim, b.window, b.kv_from) == (7, 12, 9, 2)
    assert {n for *_, n in d.all_tensors()} == set(W)  # nothing is left over, nothing is made up


def test_unknown_parts_are_refused():
    cfg = zc.config([zc.wkv()])
    shape = lambda n: zc.weights(cfg)[n].shape  # noqa: E731
    for key, value, what in (("type", "mystery", "mixer type"), ("mlp", {"kind": "sparse", "ff": 4}, "feed-forward")):
        bad = copy.deepcopy(cfg)
        bad["layers"][0][key] = value
        with pytest.raises(ValueError, match=what):
            registry.describe(bad, shape)


def test_window_rule():
    v = Z.window_visible(6, 3)
    assert v[4].tolist() == [False, False, True, True, True, False] and v[1].tolist() == [True, True] + [False] * 4
    assert Z.window_visible(5, 1).sum() == 5 and Z.window_visible(5, 99).sum() == 15


def test_rotation_turns_pairs_and_keeps_relative_positions():
    rot = {"base": 50.0, "dims": 6}
    f, mag = Z.yarn_frequencies(6, 50.0)
    assert mag == 1 and np.allclose(f, 50.0 ** (-np.arange(3) / 3))
    x = np.random.default_rng(0).standard_normal((4, 8))
    y = Z.rotate_half(x, np.arange(4), rot)
    assert np.allclose(y[0], x[0]) and np.allclose(y[:, 6:], x[:, 6:])  # position 0 and what lies behind the rotated part
    assert np.allclose(np.hypot(y[:, :3], y[:, 3:6]), np.hypot(x[:, :3], x[:, 3:6]))
    q, k = np.tile(x[:1], (9, 1)), np.tile(x[1:2], (9, 1))
    s = Z.rotate_half(q, np.arange(9), rot) @ Z.rotate_half(k, np.arange(9), rot).T
    assert np.allclose(np.diag(s, -2), s[2, 0]) and not np.isclose(s[2, 0], s[3, 0])


def test_yarn_slows_only_slow_dimensions():
    plain, _ = Z.yarn_frequencies(32, 1e4)
    f, mag = Z.yarn_frequencies(32, 1e4, {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0})
    r = plain / f
    assert np.isclose(r[0], 1) and np.isclose(r[-1], 8) and (np.diff(r) > -1e-12).all() and np.isclose(mag, 0.1 * np.log(8) + 1)
    assert np.allclose(Z.yarn_frequencies(32, 1e4, {"factor": 1.0, "original": 1024, "fast": 32.0, "slow": 1.0})[0], plain)


def test_wkv_reads_before_it_writes():
    rng = np.random.default_rng(1)
    r, k, w = (rng.random((5, 2, 3)) for _ in range(3))
    v, u = rng.random((5, 2, 4)), rng.random((2, 3))
    o = Z.wkv_scan(r, k, v, w, u)
    for t in range(5):
        want = np.einsum("hk,hv->hv", r[t] * u * k[t], v[t])
        want = want + sum(np.einsum("hk,hv->hv", r[t] * k[j] * np.prod(w[j + 1:t], 0), v[j]) for j in range(t))
        assert np.allclose(o[t], want)


def test_hgrn2_forgets_what_it_writes_over():
    h = np.random.default_rng(2).standard_normal((6, 4)) * 9
    f = Z.hgrn2_forget(h, {"f": np.eye(4), "f.b": np.zeros(4), "lower": np.array([0, 0.25, 0.5, 1.0])})
    assert (f >= [0, 0.25, 0.5, 1.0]).all() and (f <= 1).all() and (f[:, 3] == 1).all()


def test_xielu_is_smooth_at_zero_and_has_its_two_numbers():
    z = np.array([-1e-4, 0.0, 1e-4])
    assert np.allclose(Z.xielu(z, 0.3, -0.7), z / 2, atol=1e-7)
    assert np.isclose(Z.xielu(np.array([2.0]), 0.3, 9.0)[0], np.log1p(np.exp(0.3)) * 4 + 1)
    assert np.isclose(Z.xielu(np.array([-2.0]), 9.0, 0.3)[0], (0.5 + np.log1p(np.exp(0.3))) * (np.exp(-2) + 1) - 1)


def test_oracle_is_causal_and_sees_the_previous_token():
    cfg = zc.config([zc.wkv(), zc.latent(size=5), zc.hgrn2(), zc.latent(size=3, kv_from=1, heads=2)])
    W = zc.weights(cfg)
    a = dc.tokens(cfg, 24)
    b = a.copy()
    b[15] = b[15] % (cfg["vocab"] - 1) + 1
    x, y = Z.forward(cfg, W, a), Z.forward(cfg, W, b)
    assert np.allclose(x[:15], y[:15]) and all(not np.allclose(x[i], y[i]) for i in (15, 16, 23))
