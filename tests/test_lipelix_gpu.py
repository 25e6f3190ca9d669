"""The Lipelix design on the GPU against the plain oracle (oracle/lipelix_ref.py): mechanisms alone and together, prompts,
decoding, portions, mixed batches, pages and slots used again, far keys, edges of windows and kept tokens, sinks, the scheduler
and generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import decoder_cases as dc
import lipelix_cases as lc
from jgpt_b200 import ContinuousBatcher, binding
from jgpt_b200 import decoder as D
from oracle import lipelix_ref as L

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL, BF16_TOL = 1e-5, 0.04
DTYPES = ["float32", "bfloat16"]

CASES = {
    "all": lc.config([lc.att(), lc.gen(), lc.win(), lc.gen(heads=2, dim=33, mlp=lc.dense(30)), lc.att(heads=2, kv_heads=2, rot_dims=8)]),
    "order": lc.config([lc.gen(heads=1, dim=64), lc.att(v_mix=False, mlp=None), lc.win(heads=8, kv_heads=1, dim=32, vdim=32, keep=40, size=30, rot_dims=10),
                        lc.att(heads=4, kv_heads=4, dim=16, vdim=8, base=1e4), lc.win(mlp=None, v_mix=False, keep=0, size=1), lc.gen(heads=6, dim=16)],
                       width=96, vocab=128, mult=1.3, scale=0.7),
    "ragged_sizes": lc.config([lc.win(heads=5, kv_heads=5, dim=10, vdim=13, rot_dims=6, size=64, keep=16, mlp=lc.dense(21)), lc.gen(heads=3, dim=9),
                               lc.att(heads=13, kv_heads=13, dim=9, vdim=5, rot_dims=2, mlp=lc.dense(37)), lc.att(heads=1, kv_heads=1, dim=6, vdim=65)],
                              width=77, vocab=93, mult=0.3, scale=5.0),
    "large_heads": lc.config([lc.att(heads=24, kv_heads=2, dim=128, vdim=64, mlp=lc.dense(200)), lc.win(heads=20, kv_heads=1, dim=96, vdim=128, size=100, keep=17),
                              lc.gen(heads=2, dim=128), lc.win(heads=2, kv_heads=1, dim=200, vdim=256, rot_dims=64, v_mix=False, mlp=None, size=33, keep=33),
                              lc.gen(heads=1, dim=200)], width=128),
}


@pytest.fixture(scope="module")
def cases():
    return {k: lc.Case(c, seed=i) for i, (k, c) in enumerate(CASES.items())}


def _close(got, want, dtype, tol=None):
    e = dc.error(got, want)
    assert np.isfinite(e).all() and e.max() < (tol or (F32_TOL if dtype == "float32" else BF16_TOL)), (dtype, e.max(), int(e.argmax()))


# ---- the model against the oracle --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_prompt_matches_the_oracle(ctx, cases, name, dtype):
    c = cases[name]
    m = c.model(ctx, dtype)
    pool = m.newPool(60, 3)
    for n in (1, 2, 63, 131, 333):
        t = dc.tokens(c.cfg, n, n)
        _close(dc.run_steps(m, pool, [[("a", t)]])["a"], c.ref(t), dtype)
    pool.close(), m.close()


@pytest.mark.parametrize("name", ["order", "ragged_sizes"])
def test_residual_after_every_layer(ctx, cases, name):
    c = cases[name]
    m = c.model(ctx, "float32")
    pool = m.newPool(8, 1)
    t = dc.tokens(c.cfg, 37)
    got, want = m.captureLayers(t.size), []
    dc.run_steps(m, pool, [[("a", t)]])
    L.forward(c.cfg, c.W, t, want)
    for g, w in zip(got, want):
        assert np.abs(g - w).max() < 1e-5 * np.abs(w).max()
    pool.close(), m.close()


# ---- each mechanism alone ----------------------------------------------------------------------------------
def _alone(ctx, layers, dtype, sizes=(200, 1, 2, 40, 7, 50), width=64, edit=None, seed=3, tol=0.04):
    """What a layer (the last one) adds to the residual, in portions."""
    layers = layers if isinstance(layers, list) else [layers]
    c = lc.Case(lc.config(layers, width=width, mult=1.0), seed, edit)
    m = c.model(ctx, dtype, max(sizes))
    n = sum(sizes)
    pool = m.newPool(-(-n // 16), 1)
    t, want, got = dc.tokens(c.cfg, n, 5), [], []
    seq = pool.seq_alloc()
    for part in dc.cut(t, list(sizes)):
        cap = m.captureLayers(len(part))
        m.step(pool, [seq], [part], want_logits=False)
        got.append(cap)
    L.forward(c.cfg, c.W, t, want)
    front = want[-2] if len(layers) > 1 else c.W["embed"][t].astype(np.float64) * c.cfg["embedding"]["scale"]
    d, size = np.concatenate(got, 1)[-1] - want[-1], want[-1] - front
    if dtype == "float32":
        assert np.abs(d).max() < 1e-5 * np.abs(size).max()
    else:
        e = np.sqrt((d * d).mean(-1) / (size * size).mean())
        assert e.max() < tol, (e.max(), int(e.argmax()))
    pool.close(), m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [dict(), dict(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2), dict(heads=33, kv_heads=1, dim=16, vdim=24),
                                dict(dim=128, vdim=128, rot_dims=128), dict(dim=90, vdim=33, rot_dims=50), dict(dim=60, vdim=30, rot_dims=28),
                                dict(heads=2, dim=130, vdim=190, rot_dims=20), dict(heads=16, kv_heads=16, dim=31, vdim=60, rot_dims=6)])
def test_attention_on_normed_rows_alone(ctx, kw, dtype):
    _alone(ctx, lc.att(mlp=None, **kw), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [dict(), dict(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2, size=1, keep=1), dict(heads=33, kv_heads=1, dim=16, vdim=24, size=50, keep=0),
                                dict(dim=128, vdim=128, rot_dims=128, size=64, keep=64), dict(dim=90, vdim=33, rot_dims=50, size=16, keep=130),
                                dict(dim=60, vdim=30, rot_dims=28, size=17, keep=15), dict(heads=2, dim=130, vdim=190, rot_dims=20, size=150, keep=33),
                                dict(dim=96, vdim=64, size=2, keep=16), dict(size=10 ** 6, keep=10 ** 6), dict(size=65, keep=1)])
def test_windowed_attention_alone(ctx, kw, dtype):
    _alone(ctx, lc.win(mlp=None, **kw), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_heads_that_are_tiny_and_weights_that_stand_out(ctx, dtype):
    """Norm weights that differ by orders between the elements of a row and between heads; rows and heads whose size eps matters to."""
    def rows(W):
        for n, k in (("q", 120), ("k", 40)):
            W[f"l0.mix.{n}.norm"] = np.exp(np.linspace(-2, 1.0, k))[np.random.default_rng(k).permutation(k)]
            W["l0.mix." + n] = W["l0.mix." + n] * 2e-3
            W["l0.mix." + n][:20] *= 4.0  # one head is larger than the others: the norm is not the heads' own

    def heads(W):
        for n in "qk":
            W["l0.mix." + n] = W["l0.mix." + n] * 2e-3
    _alone(ctx, lc.att(mlp=None), dtype, edit=rows)
    _alone(ctx, lc.win(mlp=None), dtype, edit=heads)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("at", [-20.0, 3.0, 7.0, 11.0])
def test_learned_sinks_stand_out(ctx, dtype, at):
    """Sinks as large as hundreds of scores together, much larger, and absent; different from head to head."""
    def edit(W):
        W["l0.mix.sink"] = at + np.array([0.0, 1.5, -1.5, 0.5, -0.5, 1.0])
    _alone(ctx, lc.att(mlp=None), dtype, edit=edit, sizes=(400, 1, 2, 40, 7, 50))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("factor", [0.01, 4.0, -4.0])
def test_zero_sinks_stand_out(ctx, dtype, factor):
    """Few keys whose scores are all near 0, or spread far to both sides of it."""
    _alone(ctx, lc.win(mlp=None, size=3, keep=1, scale=factor * 14 ** -0.5), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("second", [lc.att(mlp=None), lc.win(mlp=None), lc.att(heads=12, kv_heads=4, vdim=6, mlp=None), lc.win(heads=1, kv_heads=1, dim=40, vdim=24, mlp=None),
                                    lc.att(heads=4, kv_heads=2, dim=90, vdim=12, mlp=None)])
@pytest.mark.parametrize("share", [1.0, 0.4, -2.0])
def test_values_mixed_with_the_first_ones(ctx, dtype, second, share):
    def edit(W):
        W["l2.mix.vmix"] = np.array(share)
    _alone(ctx, [lc.win(mlp=None), lc.att(v_mix=False, mlp=None), second], dtype, edit=edit)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim", [(1, 8), (3, 40), (2, 64), (2, 100), (5, 17), (1, 128), (1, 192), (1, 256), (20, 16)])
def test_general_delta_alone(ctx, heads, dim, dtype):
    _alone(ctx, lc.gen(heads, dim), dtype, sizes=(200, 1, 2, 40, 7, 31, 33, 50))


@pytest.mark.parametrize("heads,dim", [(1, 8), (3, 40), (2, 64), (2, 100), (1, 128), (1, 192), (1, 256)])
def test_general_delta_in_chunks_in_fp32(ctx, heads, dim, monkeypatch):
    """The chunked form against the oracle at fp32 accuracy, from states that earlier portions left."""
    monkeypatch.setenv("JGPT_B200_REC_CHUNK_EXACT", "1")
    _alone(ctx, lc.gen(heads, dim), "float32", sizes=(37, 64, 1, 129, 32, 200))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["forgets", "remembers", "same_key", "tiny_keys"])
def test_general_delta_extremes(ctx, which, dtype):
    def edit(W):
        if which == "forgets":
            W["l0.mix.w0"], W["l0.mix.a.b"] = W["l0.mix.w0"] + 20, W["l0.mix.a.b"] + 6
        if which == "remembers":  # nothing decays, nothing is removed: the sum of hundreds of tokens
            W["l0.mix.w0"], W["l0.mix.a.b"] = W["l0.mix.w0"] - 30, W["l0.mix.a.b"] - 30
        if which == "same_key":  # all tokens' keys point the same way: the removals depend on one another
            k = W["l0.mix.k"]
            W["l0.mix.k"] = 0.05 * k
            W["embed"] = W["embed"] * 0.3 + 1.0
        if which == "tiny_keys":
            W["l0.mix.k"] = W["l0.mix.k"] * 5e-4
    _alone(ctx, lc.gen(2, 24), dtype, edit=edit, sizes=(300, 1, 1, 50), tol=0.08)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff", [(64, 8), (77, 75), (200, 300), (1032, 24)])
def test_feed_forward_shift_and_gates_alone(ctx, width, ff, dtype):
    """Shifts of every size, gates wide open and shut, a feed-forward part; batches large enough for every product kernel."""
    def edit(W):
        W["l0.shift"] = np.linspace(-1.5, 2.5, width)
        W["l0.rg1.b"], W["l0.rg2.b"] = np.linspace(-8, 8, width), np.linspace(6, -6, width)
        W["l0.norm1b"] = np.exp(np.linspace(-1, 1, width))
    _alone(ctx, lc.gen(2, 8, mlp=lc.dense(ff)), dtype, sizes=(300, 1, 2, 3, 20, 64, 128, 90), width=width, edit=edit)


# ---- how a sequence is cut must not matter -------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[1], [2], [3, 2, 7], [16], [17], [64, 1, 1, 2], [150, 1]])
def test_portions_equal_the_whole(ctx, cases, sizes, dtype):
    for name in ("order", "ragged_sizes"):
        c = cases[name]
        m = c.model(ctx, dtype)
        pool = m.newPool(24, 2)
        t = dc.tokens(c.cfg, 190, 3)
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), dtype)
        pool.close(), m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(ctx, cases, dtype):
    c = cases["all"]
    m = c.model(ctx, dtype)
    pool = m.newPool(40, 1)
    t = dc.tokens(c.cfg, 500, 4)
    _close(dc.run_steps(m, pool, [[("a", t[:20])]] + [[("a", t[i:i + 1])] for i in range(20, 500)])["a"], c.ref(t), dtype)
    pool.close(), m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_mixed_batches_with_blocks_and_slots_used_again(ctx, cases, name, dtype):
    """Nine requests through three slots and a pool that holds far fewer blocks than they need together, on storage that
    starts as NaN patterns: what a request reads, it or nobody has written."""
    from jgpt_b200 import binding as B
    c = cases[name]
    m = c.model(ctx, dtype)
    pool = m.newPool(40, 3)
    p, n = pool.storage()
    B.check(m._lib.jgpt_dev_memset(ctx.handle, p, 0xFF, n))
    toks = {f"r{i}": dc.tokens(c.cfg, n, 50 + i) for i, n in enumerate([1, 150, 33, 200, 64, 17, 2, 180, 90])}
    got = dc.run_steps(m, pool, dc.mixed_plan(toks, 7))
    for r, t in toks.items():
        _close(got[r], c.ref(t), dtype)
    assert pool.free_blocks() == 40
    pool.close(), m.close()


def test_batch_of_unequal_requests_equals_each_alone(ctx, cases):
    c = cases["all"]
    m = c.model(ctx, "bfloat16", max_rows=1600)
    pool = m.newPool(160, 9)
    toks = {f"r{i}": dc.tokens(c.cfg, n, 80 + i) for i, n in enumerate([5, 1, 64, 130, 2, 17, 700, 600])}  # blocks of several rows in the norms
    together = dc.run_steps(m, pool, [list(toks.items())])
    for r, t in toks.items():
        alone = dc.run_steps(m, pool, [[(r, t)]])[r]
        assert dc.error(together[r], alone.astype(np.float64)).max() < 0.02
        _close(together[r], c.ref(t), "bfloat16")
    pool.close(), m.close()


def test_many_rows_in_a_step(ctx, cases):
    """Enough rows for blocks of several rows everywhere, entries that start and end inside them."""
    c = cases["all"]
    m = c.model(ctx, "bfloat16", max_rows=9600)
    sizes = [150, 1, 333, 2, 90] * 15 + [700]
    pool = m.newPool(sum(-(-n // 16) for n in sizes), len(sizes))
    base = {n: dc.tokens(c.cfg, n, n) for n in set(sizes)}
    got = dc.run_steps(m, pool, [[(f"r{i}", base[n]) for i, n in enumerate(sizes)]])
    for i, n in enumerate(sizes):
        _close(got[f"r{i}"], c.ref(base[n]), "bfloat16")
    pool.close(), m.close()


def test_decode_batches_of_many_sequences(ctx, cases):
    """Steps of single tokens at every length of a page, as many sequences as take another split of the keys, replayed graphs."""
    c = cases["large_heads"]
    m = c.model(ctx, "bfloat16")
    for n in (1, 5, 40, 140):
        pool = m.newPool(n * 12, n)
        toks = [dc.tokens(c.cfg, 60 + 7 * (i % 17), 500 + i) for i in range(n)]
        seqs = [pool.seq_alloc() for _ in range(n)]
        for i in range(0, n, 3):
            m.step(pool, seqs[i:i + 3], [t[:-20] for t in toks[i:i + 3]], want_logits=False)
        for j in range(20):
            if j % 5 == 4:
                logits, _ = m.step(pool, seqs, [t[len(t) - 20 + j:][:1] for t in toks], np.arange(n))
                for i in range(0, min(n, 40), 7):
                    _close(logits[i:i + 1], c.ref(toks[i])[len(toks[i]) - 20 + j:][:1], "bfloat16")
            else:
                lens = [len(t) - 20 + j for t in toks]
                m.forwardDecodeBatch(pool, seqs, [t[k] for t, k in zip(toks, lens)], lens, want_logits=False)
        pool.close()
    m.close()


# ---- far keys, edges, first tokens -----------------------------------------------------------------------------
def _needle(cfg, needle=1, query=2):
    """Weights of one attention layer with which a query of the `query` token falls on keys of the `needle` token alone: its
    projection is that of the needle's key; the mixer's input depends on the token only."""
    def edit(W):
        W["l0.shift"], W["l0.norm1"] = W["l0.shift"] * 0, W["l0.norm1"] * 0 + 1
        h = W["embed"].astype(np.float64) * cfg["embedding"]["scale"]
        h = h / np.sqrt((h * h).mean(-1, keepdims=True) + cfg["norm"]["eps"])
        m, n, q = cfg["layers"][0]["mixer"], h[needle], h[query]
        k = W["l0.mix.k"].reshape(m["kv_heads"], m["dim"], -1)
        k = np.repeat(k, m["heads"] // m["kv_heads"], 0).reshape(-1, cfg["width"])
        W["l0.mix.q"] = k + np.outer(k @ (n - q), q) / (q @ q)
        for x in ("q.norm", "k.norm"):
            if "l0.mix." + x in W:
                W["l0.mix." + x] = W["l0.mix." + x] * 0 + 1
        W["l0.mix.v"] = W["l0.mix.v"] + np.outer(W["l0.mix.v"] @ n, n) * 3 / (n @ n)  # and its value stands out
    return edit


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_far_key_among_hundreds(ctx, dtype):
    """A key at a sequence's start, a page's edges or just before the query decides the query's output."""
    cfg = lc.config([lc.att(heads=4, kv_heads=2, dim=64, vdim=32, rot_dims=4, base=1e5, scale=0.35, mlp=None)], mult=3.0)
    c = lc.Case(cfg, seed=6, edit=_needle(cfg))
    m = c.model(ctx, dtype, max_rows=700)
    pool = m.newPool(50, 2)
    hay = dc.tokens(cfg, 650, 1) % (cfg["vocab"] - 4) + 4
    for at in (0, 1, 15, 16, 17, 63, 64, 255, 256, 500, 640):
        t = hay.copy()
        t[at], t[641], t[649] = 1, 2, 2
        other = t.copy()
        other[at] = hay[at]
        want = c.ref(t)
        assert dc.error(c.ref(other), want)[[641, 649]].min() > 0.3  # the far key shows
        for sizes in ([650], [641, 1, 7, 1], [at + 1, 2, 3, 1, 64], [600, 50]):
            _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], want, dtype)
    pool.close(), m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep", [(37, 5), (130, 20), (64, 16), (16, 33), (100, 0), (1, 3), (80, 64)])
def test_edges_of_windows_and_kept_tokens(ctx, dtype, size, keep):
    """One key just inside or just outside the window or the kept tokens, for queries in prompts, in portions and decoded: an edge
    that is off by one moves the output by far more than the tolerance."""
    cfg = lc.config([lc.win(heads=4, kv_heads=2, dim=64, vdim=32, rot_dims=4, base=1e5, scale=0.4, size=size, keep=keep, mlp=None)], mult=3.0)
    c = lc.Case(cfg, seed=6, edit=_needle(cfg))
    m = c.model(ctx, dtype, max_rows=400)
    pool = m.newPool(30, 2)
    hay = dc.tokens(cfg, 330, 1) % (cfg["vocab"] - 4) + 4
    for p in (size + keep + 3, 207, 256, 300):
        for at in sorted({p - size, p - size + 1, keep - 1, keep, p}):
            if at < 0:
                continue
            t = hay[:p + 9].copy()
            t[p] = 2
            if at < p:
                t[at] = 1
            want = c.ref(t)
            if at < p:  # the oracle tells the edge apart
                off = [{**cfg, "layers": [lc.win(heads=4, kv_heads=2, dim=64, vdim=32, rot_dims=4, base=1e5, scale=0.4, size=s, keep=k, mlp=None)]}
                       for s, k in ((size + (1 if at == p - size else -1), keep),) if at in (p - size, p - size + 1) and at >= keep and s > 0]
                off += [{**cfg, "layers": [lc.win(heads=4, kv_heads=2, dim=64, vdim=32, rot_dims=4, base=1e5, scale=0.4, size=size, keep=k, mlp=None)]}
                        for k in ((keep + (1 if at == keep else -1)),) if at in (keep - 1, keep) and at <= p - size]
                for o in off:
                    assert dc.error(L.forward(o, c.W, t), want)[p] > 0.2
            for sizes in ([p + 9], [p, 1, 1, 7], [max(p - 3, 1), 2, 2, 20], [max(p - 40, 1), 100]):
                _close(dc.run_steps(m, pool, [[("a", x)] for x in dc.cut(t, sizes)])["a"], want, dtype)
    pool.close(), m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(ctx, cases, dtype):
    """Sequences of one to five tokens, whole and token by token, in slots that longer ones have left."""
    c = cases["all"]
    m = c.model(ctx, dtype)
    pool = m.newPool(6, 1)
    dc.run_steps(m, pool, [[("x", dc.tokens(c.cfg, 90, 9))]])
    for n in range(1, 6):
        t = dc.tokens(c.cfg, n, 70 + n)
        for sizes in ([n], [1], [2, 1]):
            _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), dtype)
    pool.close(), m.close()


def test_positions_far_from_the_start(ctx):
    """Rotations of large positions against float64 angles, a long state."""
    cfg = lc.config([lc.att(base=50.0, heads=2, mlp=None), lc.win(base=60.0, heads=2, kv_heads=2, size=300, mlp=None), lc.gen(1, 12)])
    c = lc.Case(cfg, seed=2)
    m = c.model(ctx)
    pool = m.newPool(160, 1)
    t = dc.tokens(cfg, 1500, 6)
    _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, [500])])["a"], c.ref(t), "float32")
    pool.close(), m.close()


# ---- scheduler, generation -----------------------------------------------------------------------------------
def test_greedy_generation_equals_the_oracle(ctx, cases):
    c = cases["ragged_sizes"]
    m = c.model(ctx, "float32", max_rows=16)
    for i, n in enumerate([1, 5, 40]):  # the longest prompt goes in as portions
        prompt = dc.tokens(c.cfg, n, 200 + i)
        want, margin = dc.greedy(c, prompt, 12)
        assert margin > 1e-4
        got = m.generateGpuKv(prompt, 12)
        assert got[n:n + len(want)].tolist() == want and (got[n + len(want):] == 0).all()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_continuous_batching(ctx, cases, dtype):
    c = cases["all"]
    m = c.model(ctx, dtype, max_rows=24)
    pool = m.newPool(18, 5)
    batch = ContinuousBatcher(m, pool, max_running=4)
    prompts = [dc.tokens(c.cfg, n, 300 + i) for i, n in enumerate([3, 60, 1, 25, 100, 8, 30])]
    ids = [batch.submit(p, 10) for p in prompts]
    batch.run(500)
    for p, r in zip(prompts, ids):
        got, state, _ = batch.result(r)
        assert state == 2
        if dtype == "float32":
            want, margin = dc.greedy(c, p, 10)
            assert margin < 1e-4 or got.tolist() == want
        else:
            lg = L.forward(c.cfg, c.W, np.concatenate([p, got]))  # every pick is near the oracle's best
            for j, tok in enumerate(got):
                row = lg[len(p) - 1 + j]
                assert row.max() - row[tok] < 0.1 * row.std()
    batch.close(), pool.close(), m.close()


def test_misfits_are_refused(ctx):
    def build(*layers):
        lc.Case(lc.config(list(layers))).model(ctx).close()
    for layers in ((lc.att(), lc.win(vdim=16)), (lc.win(size=-1),), (lc.att(dim=8, rot_dims=10),), (lc.gen(dim=257),), (lc.win(size=0, keep=3),)):
        with pytest.raises((ValueError, binding.JgptError)):  # values of another size, a window of nothing, more turned than there is, heads too large
            build(*layers)
    m = lc.Case(lc.config([lc.att()])).model(ctx)
    with pytest.raises(ValueError):
        m.setTensor(0, 0, D.W_VMIX, np.ones(1))  # the values' source has no share
    m.close()


def test_command_lines(ctx, cases, tmp_path):
    from jgpt_b200 import safetensors

    c = cases["all"]
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir(), out.mkdir()
    json.dump(c.cfg, open(folder / "config.json", "w"))
    safetensors.write_bf16(folder / "model.safetensors", c.W)
    t = [int(x) for x in dc.tokens(c.cfg, 40, 2)]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:33], "want": [32, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": t[33:], "want": [6]}, {"id": "b", "tokens": t[:2], "want": []}], "end": ["a", "b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    want = c.ref(t)
    _close(np.fromfile(out / "0.f32", np.float32).reshape(2, -1), want[[32, 3]], "float32")
    _close(np.fromfile(out / "1.f32", np.float32).reshape(1, -1), want[[39]], "float32")
    r = subprocess.run([sys.executable, "-m", "jgpt_b200.generate", "--model", str(folder), "--dtype", "float32", "--prompt", ",".join(map(str, t[:5])),
                        "--max-new", "6"], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    line = json.loads([x for x in r.stdout.splitlines() if x.startswith("{")][0])
    assert line["tokens"] == dc.greedy(c, t[:5], 6)[0]
