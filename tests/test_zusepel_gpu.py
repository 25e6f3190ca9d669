"""The Zusepel design on the GPU against the plain oracle (oracle/zusepel_ref.py): mechanisms alone and together, prompts,
decoding, portions, mixed batches, pages and slots used again, window edges, shared caches, the scheduler and generation."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import decoder_cases as dc
import zusepel_cases as zc
from jgpt_b200 import ContinuousBatcher
from jgpt_b200 import decoder as D
from oracle import hybrid_ref as R
from oracle import zusepel_ref as Z

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL, BF16_TOL = 3e-5, 0.06
DTYPES = ["float32", "bfloat16"]

CASES = {
    "all": zc.config([zc.hgrn2(), zc.wkv(), zc.latent(), zc.latent(kv_from=2, size=25, heads=2, vdim=16)]),
    "order": zc.config([zc.latent(ff=0, size=70), zc.wkv(heads=5, dim=16, ff=0), zc.latent(kv_from=0, size=90), zc.hgrn2(heads=1, dim=40, vdim=12, ff=33),
                        zc.latent(kv_rank=60, rot_dim=8, yarn=None, base=1e4), zc.latent(kv_from=4, kv_rank=60, rot_dim=8, yarn=None, base=1e4, ff=0)],
                       width=96, vocab=128, mult=1.0),
    "ragged_sizes": zc.config([zc.wkv(heads=1, dim=33, ff=50), zc.latent(heads=5, dim=9, rot_dim=6, vdim=11, q_rank=19, kv_rank=23, size=17, ff=37),
                               zc.hgrn2(heads=3, dim=7, vdim=9, ff=21)], width=77, vocab=93, mult=0.37),
    "large_heads": zc.config([zc.latent(heads=20, dim=64, rot_dim=32, vdim=48, q_rank=96, kv_rank=300, size=50), zc.wkv(heads=1, dim=128),
                              zc.hgrn2(heads=2, dim=128, vdim=160), zc.latent(heads=2, dim=150, rot_dim=64, vdim=190, q_rank=40, kv_rank=500, size=200),
                              zc.latent(heads=1, dim=100, rot_dim=48, vdim=64, q_rank=40, kv_rank=160, size=20)], width=128),
}


@pytest.fixture(scope="module")
def cases():
    return {k: zc.Case(c, seed=i) for i, (k, c) in enumerate(CASES.items())}


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
    m = c.model(ctx)
    pool = m.newPool(8, 1)
    t = dc.tokens(c.cfg, 37)
    got, want = m.captureLayers(t.size), []
    dc.run_steps(m, pool, [[("a", t)]])
    Z.forward(c.cfg, c.W, t, want)
    for g, w in zip(got, want):
        assert np.abs(g - w).max() < 2e-5 * np.abs(w).max()
    pool.close(), m.close()


# ---- each mechanism alone ----------------------------------------------------------------------------------
def _alone(ctx, layer, dtype, apply, n=150, width=64, names=None, tol=0.03):
    """x + mixer(RMS(x)) [+ ff] in a model without layer scales and depth averages, portions [n - 40, 1, 2, 37]."""
    cfg = zc.config([layer], width=width)
    W = zc.weights(cfg, 3)
    from jgpt_b200 import registry
    y = registry.describe(cfg, lambda k: W[k].shape).layers[0]
    drop = (D.W_LS1, D.W_LS2, D.W_DWA)
    y.tensors = {k: v for k, v in y.tensors.items() if k not in drop}
    top = D.DecoderConfig(101, width, D.NO_LIMIT, 1e-5, [y], pos_table=False, norm=D.NORM_RMS,
                          tensors={D.W_EMBED: "embed", D.W_FINAL_NORM: "final.norm"})
    m = D.DecoderModel(ctx, top, dtype, 160)
    m.loadTensors(W.__getitem__)
    pool = m.newPool(-(-n // 16), 1)
    t = dc.tokens(cfg, n, 5)
    seq, got = pool.seq_alloc(), []
    for part in dc.cut(t, [n - 40, 1, 2, 37]):
        cap = m.captureLayers(len(part))
        m.step(pool, [seq], [part], want_logits=False)
        got.append(cap[0])
    x = W["embed"][t].astype(np.float64)
    L = R.sub({k: np.asarray(v, np.float64) for k, v in W.items()}, "l0.")
    want = apply(x, L)
    got = np.concatenate(got) - x
    if dtype == "float32":
        assert np.abs(got - want).max() < 2e-5 * np.abs(want).max()
    else:  # a head whose sum nearly cancels is normed all the same: single values may be far off after rounding
        assert np.sqrt(((got - want) ** 2).mean()) < tol * np.sqrt((want ** 2).mean())
    pool.close(), m.close()


def _mixer(fn, layer):
    return lambda x, L: fn(R.rms_norm(x, L["norm1"], 1e-5), R.sub(L, "mix."), layer["mixer"], 1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim", [(1, 8), (3, 40), (2, 64), (2, 100)])
def test_wkv_alone(ctx, heads, dim, dtype):
    layer = zc.wkv(heads, dim, ff=0)
    _alone(ctx, layer, dtype, _mixer(Z.wkv_mixer, layer))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(1, 5, 16), (3, 48, 40), (2, 128, 64), (2, 30, 200)])
def test_hgrn2_alone(ctx, heads, dim, vdim, dtype):
    layer = zc.hgrn2(heads, dim, vdim, ff=0)
    _alone(ctx, layer, dtype, _mixer(Z.hgrn2_mixer, layer))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [dict(), dict(heads=17, size=1), dict(yarn=None, size=64), dict(dim=128, rot_dim=64, vdim=128, kv_rank=512, size=1000),
                                dict(heads=1, dim=40, rot_dim=2, vdim=72, kv_rank=130, size=77)])
def test_latent_attention_alone(ctx, kw, dtype):
    layer = zc.latent(ff=0, **kw)
    _alone(ctx, layer, dtype, _mixer(lambda h, W, m, e: Z.latent_attention(h, W, m, e, Z.latent_keys(h, W, m, e)), layer))


@pytest.mark.parametrize("dtype", DTYPES)
def test_unbounded_window_and_partly_rotated_heads(ctx, dtype):
    """No mask: everything before the query; only the first rot.dims of the rotated part turn."""
    layer = zc.latent(ff=0, rot_dim=14, size=10 ** 6)
    layer["mixer"]["rot"]["dims"] = 8
    _alone(ctx, layer, dtype, _mixer(lambda h, W, m, e: Z.latent_attention(h, W, m, e, Z.latent_keys(h, W, m, e)), layer))
    free = copy.deepcopy(layer)
    del free["mixer"]["mask"]
    _alone(ctx, free, dtype, _mixer(lambda h, W, m, e: Z.latent_attention(h, W, layer["mixer"], e, Z.latent_keys(h, W, m, e)), free))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [8, 75, 200])
def test_xielu_alone(ctx, ff, dtype):
    layer = zc.hgrn2(1, 4, 4, ff=ff)

    def apply(x, L):
        y = Z.hgrn2_mixer(R.rms_norm(x, L["norm1"], 1e-5), R.sub(L, "mix."), layer["mixer"], 1e-5)
        z = R.linear(R.rms_norm(x + y, L["norm2"], 1e-5), L["mlp.up"])
        return y + R.linear(Z.xielu(z, *L["mlp.act"]), L["mlp.down"])
    _alone(ctx, layer, dtype, apply)


@pytest.mark.parametrize("dtype", DTYPES)
def test_depth_averages_and_layer_scales_stand_out(ctx, dtype):
    """The last layer hands on the embedding and the first layer's result only; a scale of zero takes a part out."""
    def edit(W):
        W["l3.dwa"] = np.array([0.7, -1.2, 0.0, 0.0, 0.25])
        W["l1.ls2"] = W["l1.ls2"] * 0
        W["l2.ls1"] = W["l2.ls1"] * np.where(np.arange(72) % 2, 3.0, 0.0)
    c = zc.Case(CASES["all"], seed=8, edit=edit)
    m = c.model(ctx, dtype)
    pool = m.newPool(10, 1)
    t = dc.tokens(c.cfg, 140, 1)
    for sizes in ([140], [100, 1, 39]):
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), dtype)
    pool.close(), m.close()


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


@pytest.mark.parametrize("least", ["2", "20", "0"])
@pytest.mark.parametrize("name", list(CASES))
def test_latent_forms_agree(ctx, cases, name, least, monkeypatch):
    """Portions on the latents themselves and with keys and values written out, from every length on and never."""
    monkeypatch.setenv("JGPT_B200_LATENT_EXPAND_MIN", least)
    c = cases[name]
    m = c.model(ctx, "bfloat16")
    pool = m.newPool(60, 3)
    t = dc.tokens(c.cfg, 230, 17)
    for sizes in ([230], [2, 3, 70, 1, 19, 20, 21, 64], [129, 1, 100]):
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), "bfloat16")
    toks = {f"r{i}": dc.tokens(c.cfg, L, 50 + i) for i, L in enumerate([1, 150, 33, 64, 17, 2])}
    got = dc.run_steps(m, pool, dc.mixed_plan(toks, 3))
    for r, x in toks.items():
        _close(got[r], c.ref(x), "bfloat16")
    pool.close(), m.close()


def test_written_out_keys_in_several_batches(ctx, cases):
    """Prompts whose keys do not fit the workspace together, and one whose window does not fit it at all."""
    c = cases["order"]
    m = c.model(ctx, "bfloat16", max_rows=80)  # room for 160 keys at a time
    pool = m.newPool(60, 3)
    t, u = dc.tokens(c.cfg, 320, 4), dc.tokens(c.cfg, 300, 5)
    plan = [[("a", t[:80])], [("b", u[:70])], [("a", t[80:150]), ("b", u[70:72])], [("b", u[72:140])], [("a", t[150:230])], [("a", t[230:231]), ("b", u[140:205])],
            [("b", u[205:270])], [("a", t[231:300])]]
    got = dc.run_steps(m, pool, plan)
    _close(got["a"], c.ref(t[:300]), "bfloat16"), _close(got["b"], c.ref(u[:270]), "bfloat16")
    pool.close(), m.close()


@pytest.mark.parametrize("name", list(CASES))
def test_chunked_recurrences_at_full_precision(ctx, cases, name, monkeypatch):
    monkeypatch.setenv("JGPT_B200_REC_CHUNK_EXACT", "1")
    monkeypatch.setenv("JGPT_B200_REC_CHUNK_MIN", "6")
    c = cases[name]
    m = c.model(ctx, "float32")
    pool = m.newPool(60, 3)
    t = dc.tokens(c.cfg, 320, 17)
    for sizes in ([320], [6], [5, 7, 1, 40, 2, 16, 17, 33], [161, 1, 158]):
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), "float32")
    toks = {f"r{i}": dc.tokens(c.cfg, L, 50 + i) for i, L in enumerate([1, 150, 33, 64, 17, 2])}
    got = dc.run_steps(m, pool, dc.mixed_plan(toks, 3))
    for r, x in toks.items():
        _close(got[r], c.ref(x), "float32")
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
    toks = {f"r{i}": dc.tokens(c.cfg, L, 50 + i) for i, L in enumerate([1, 150, 33, 200, 64, 17, 2, 180, 90])}
    got = dc.run_steps(m, pool, dc.mixed_plan(toks, 7))
    for r, t in toks.items():
        _close(got[r], c.ref(t), dtype)
    assert pool.free_blocks() == 40
    pool.close(), m.close()


def test_batch_of_unequal_requests_equals_each_alone(ctx, cases):
    c = cases["all"]
    m = c.model(ctx, "bfloat16")
    pool = m.newPool(80, 6)
    toks = {f"r{i}": dc.tokens(c.cfg, L, 80 + i) for i, L in enumerate([5, 1, 64, 130, 2, 17])}
    together = dc.run_steps(m, pool, [list(toks.items())])
    for r, t in toks.items():
        alone = dc.run_steps(m, pool, [[(r, t)]])[r]
        assert dc.error(together[r], alone.astype(np.float64)).max() < 0.03
        _close(together[r], c.ref(t), "bfloat16")
    pool.close(), m.close()


def test_decode_batches_of_many_sequences(ctx, cases):
    """Steps of single tokens at every length of a page, as many sequences as take another split of the keys, replayed graphs."""
    c = cases["large_heads"]
    m = c.model(ctx, "bfloat16")
    for n in (1, 5, 40):
        pool = m.newPool(n * 8, n)
        toks = [dc.tokens(c.cfg, 60 + 3 * (i % 17), 500 + i) for i in range(n)]
        seqs = [pool.seq_alloc() for _ in range(n)]
        for i in range(0, n, 4):
            m.step(pool, seqs[i:i + 4], [t[:-20] for t in toks[i:i + 4]], want_logits=False)
        for j in range(20):
            logits = None
            if j % 5 == 4:
                logits, _ = m.step(pool, seqs, [t[len(t) - 20 + j:][:1] for t in toks], np.arange(n))
            else:
                lens = [len(t) - 20 + j for t in toks]
                m.forwardDecodeBatch(pool, seqs, [t[k] for t, k in zip(toks, lens)], lens, want_logits=False)
            if logits is not None:
                for i in range(0, n, 7):
                    _close(logits[i:i + 1], c.ref(toks[i])[len(toks[i]) - 20 + j:][:1], "bfloat16", 0.08)
        pool.close()
    m.close()


# ---- edges -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("size", [1, 2, 15, 16, 17, 31, 33, 64, 100])
def test_window_edges_stand_out(ctx, size):
    """Scores are large enough for a query's weight to sit on few keys: a key too many or too few at the window's or a page's
    edge changes the logits, shown on the oracle itself with windows one token longer and shorter.  The second layer reads the
    first one's cache through another window."""
    cfg = zc.config([zc.latent(size=size, scale=0.35, ff=0), zc.latent(size=size + 9 if size < 90 else size - 33, scale=0.35, kv_from=0, heads=2, ff=0)], mult=1.5)
    c = zc.Case(cfg, seed=size)
    t = dc.tokens(cfg, 210, size)
    want = c.ref(t)
    for layer, by in ((0, 1), (0, -1), (1, 1), (1, -1)):
        wrong = copy.deepcopy(cfg)
        wrong["layers"][layer]["mixer"]["mask"]["size"] += by
        if wrong["layers"][layer]["mixer"]["mask"]["size"] > 0:
            assert dc.error(c.ref(t, wrong), want).max() > 0.2
    for dtype in DTYPES:
        m = c.model(ctx, dtype)
        pool = m.newPool(14, 1)
        for sizes in ([210], [37, 1, 1, 30, 2], [205, 1], [1], [2]):
            e = dc.error(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], want)
            assert e.max() < (F32_TOL if dtype == "float32" else 0.12), (dtype, sizes, e.max(), int(e.argmax()))
        pool.close(), m.close()


def test_a_far_key_is_found_through_the_recurrent_states(ctx):
    """Slow decays: a token among the first shows hundreds of tokens later, whatever the cuts."""
    cfg = zc.config([zc.wkv(heads=2, dim=16), zc.hgrn2(heads=2, dim=16, vdim=16)])

    def slow(W):
        W["l0.mix.w0"] = W["l0.mix.w0"] * 0 - 8.0
        W["l1.mix.f.b"] = W["l1.mix.f.b"] * 0 + 7.0
        W["l1.mix.f"] = W["l1.mix.f"] * 0.5
    c = zc.Case(cfg, seed=3, edit=slow)
    t = dc.tokens(cfg, 600, 1)
    u = t.copy()
    u[3] = u[3] % (cfg["vocab"] - 1) + 1
    assert dc.error(c.ref(u)[-1:], c.ref(t)[-1:]).max() > 20 * F32_TOL  # the early token shows at the end
    m = c.model(ctx, "float32")
    pool = m.newPool(40, 1)
    for toks in (t, u):
        for sizes in ([512, 60, 1], [7, 2, 93]):
            _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(toks, sizes)])["a"], c.ref(toks), "float32")
    pool.close(), m.close()


def test_gates_at_their_ends(ctx, monkeypatch):
    """Channels that forget everything from one token to the next beside channels that forget nothing, a lower bound of 1."""
    monkeypatch.setenv("JGPT_B200_REC_CHUNK_EXACT", "1")
    cfg = zc.config([zc.wkv(heads=2, dim=32), zc.hgrn2(heads=2, dim=32, vdim=16)])

    def edit(W):
        W["l0.mix.w0"] = np.where(np.arange(64) % 2, 4.0, -12.0)
        W["l1.mix.f.b"] = np.where(np.arange(64) % 2, -25.0, 25.0)
        W["l1.mix.lower"] = np.where(np.arange(64) % 3 == 0, 0.0, np.where(np.arange(64) % 3 == 1, 0.5, 1.0))
    c = zc.Case(cfg, seed=4, edit=edit)
    t = dc.tokens(cfg, 200, 1)
    for dtype in DTYPES:
        m = c.model(ctx, dtype)
        pool = m.newPool(16, 1)
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, [100, 1, 99])])["a"], c.ref(t), dtype)
        pool.close(), m.close()


def test_previous_token_across_portions_and_slots(ctx):
    """Mixes that are all previous token: the first token sees zeros (not the slot's former owner), the first token of a
    portion what the last one ended with."""
    cfg = zc.config([zc.wkv(heads=2, dim=16, ff=0), zc.wkv(heads=3, dim=8, ff=0)])

    def edit(W):
        for n in W:
            if ".mu." in n:
                W[n] = W[n] * 0 + 1
    c = zc.Case(cfg, seed=9, edit=edit)
    m = c.model(ctx)
    pool = m.newPool(8, 1)
    for i, sizes in enumerate(([1], [2], [3], [1, 2, 4, 2, 1], [5], [40])):
        t = dc.tokens(cfg, 40, i)
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), "float32")
    pool.close(), m.close()


def test_positions_far_from_the_start(ctx):
    """Rotations of large positions, plain and scaled, against float64 angles."""
    cfg = zc.config([zc.latent(size=30, base=50.0), zc.latent(size=30, yarn=None, base=5e5)])
    c = zc.Case(cfg, seed=2)
    m = c.model(ctx)
    pool = m.newPool(160, 1)
    t = dc.tokens(cfg, 2500, 6)
    _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, [500])])["a"], c.ref(t), "float32")
    pool.close(), m.close()


# ---- scheduler, generation -----------------------------------------------------------------------------------
def test_greedy_generation_equals_the_oracle(ctx, cases):
    c = cases["ragged_sizes"]
    m = c.model(ctx, "float32", max_rows=16)
    for i, L in enumerate([1, 5, 40]):  # the longest prompt goes in as portions
        prompt = dc.tokens(c.cfg, L, 200 + i)
        want, margin = dc.greedy(c, prompt, 12)
        assert margin > 1e-4
        got = m.generateGpuKv(prompt, 12)
        assert got[L:L + len(want)].tolist() == want and (got[L + len(want):] == 0).all()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_continuous_batching(ctx, cases, dtype):
    c = cases["all"]
    m = c.model(ctx, dtype, max_rows=24)
    pool = m.newPool(18, 5)
    batch = ContinuousBatcher(m, pool, max_running=4)
    prompts = [dc.tokens(c.cfg, L, 300 + i) for i, L in enumerate([3, 60, 1, 25, 100, 8, 30])]
    ids = [batch.submit(p, 10) for p in prompts]
    batch.run(500)
    for p, r in zip(prompts, ids):
        got, state, _ = batch.result(r)
        assert state == 2
        if dtype == "float32":
            want, margin = dc.greedy(c, p, 10)
            assert margin < 1e-4 or got.tolist() == want
        else:
            lg = Z.forward(c.cfg, c.W, np.concatenate([p, got]))  # every pick is near the oracle's best
            for j, tok in enumerate(got):
                row = lg[len(p) - 1 + j]
                assert row.max() - row[tok] < 0.25 * row.std()
    batch.close(), pool.close(), m.close()


def test_misfits_are_refused(ctx):
    def build(layers, **kw):
        c = zc.Case(zc.config(layers, **kw))
        c.model(ctx).close()
    with pytest.raises(ValueError):  # the source has other sizes
        build([zc.latent(kv_rank=44), zc.latent(kv_rank=48, kv_from=0)])
    with pytest.raises(ValueError):  # another rotation
        build([zc.latent(base=300.0), zc.latent(base=301.0, kv_from=0)])
    with pytest.raises(ValueError):  # no cache of its own
        build([zc.latent(), zc.latent(kv_from=0), zc.latent(kv_from=1)])
    with pytest.raises(ValueError):
        build([zc.wkv(), zc.latent(kv_from=0)])


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
