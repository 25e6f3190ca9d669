"""The Nefipel design on the GPU against the plain oracle (oracle/nefipel_ref.py): mechanisms alone and together, prompts,
decoding, portions, mixed batches, pages and slots used again, far keys, the scheduler and generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import decoder_cases as dc
import nefipel_cases as nc
from jgpt_b200 import ContinuousBatcher
from jgpt_b200 import decoder as D
from jgpt_b200 import registry
from oracle import hybrid_ref as R
from oracle import nefipel_ref as N

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL, BF16_TOL = 3e-5, 0.06
DTYPES = ["float32", "bfloat16"]

CASES = {
    "both": nc.config([nc.att(), nc.diff(), nc.att(heads=2, kv_heads=2, rot_dims=8), nc.diff()]),
    "order": nc.config([nc.diff(mlp=nc.dense(50), yarn=None), nc.att(mlp=nc.moe(10, 2, 4, 3, 2)), nc.diff(mlp=None, at=0.8), nc.att(mlp=None, base=1e4),
                        nc.att(heads=8, kv_heads=1, dim=32, vdim=32), nc.diff(heads=3, kv_heads=1, mlp=nc.moe(5, 1, 5, 1, 1, ff=50, shared=0), base=900.0)],
                       width=96, vocab=128, alpha=1.0, scale=1.0),
    "ragged_sizes": nc.config([nc.diff(heads=5, kv_heads=5, dim=10, vdim=13, rot_dims=6, mlp=nc.moe(3, 2, 2, 5, 4, ff=21, shared=13)),
                               nc.att(heads=3, kv_heads=1, dim=9, vdim=11, rot_dims=2, mlp=nc.dense(37)), nc.att(heads=1, kv_heads=1, dim=6, vdim=30)],
                              width=77, vocab=93, alpha=0.6, scale=11.0),
    "large_heads": nc.config([nc.diff(heads=24, kv_heads=2, dim=64, vdim=128, mlp=nc.moe(40, 8, 6, 4, 2, ff=72, shared=80)),
                              nc.att(heads=20, kv_heads=1, dim=128, vdim=64, mlp=nc.dense(200)), nc.diff(heads=2, kv_heads=1, dim=100, vdim=200, mlp=None),
                              nc.att(heads=2, kv_heads=2, dim=200, vdim=256, rot_dims=64, mlp=None)], width=128),
}


@pytest.fixture(scope="module")
def cases():
    """Per model: natural choices of experts for float32, settled ones for bfloat16."""
    return {k: {d: nc.Case(c, seed=i, settled=d == "bfloat16") for d in DTYPES} for i, (k, c) in enumerate(CASES.items())}


def _close(got, want, dtype, tol=None):
    e = dc.error(got, want)
    assert np.isfinite(e).all() and e.max() < (tol or (F32_TOL if dtype == "float32" else BF16_TOL)), (dtype, e.max(), int(e.argmax()))


# ---- the model against the oracle --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_prompt_matches_the_oracle(ctx, cases, name, dtype):
    c = cases[name][dtype]
    m = c.model(ctx, dtype)
    pool = m.newPool(60, 3)
    for n in (1, 2, 63, 131, 333):
        t = dc.tokens(c.cfg, n, n)
        _close(dc.run_steps(m, pool, [[("a", t)]])["a"], c.ref(t), dtype)
    pool.close(), m.close()


@pytest.mark.parametrize("name", ["order", "ragged_sizes"])
def test_residual_after_every_layer(ctx, cases, name):
    c = cases[name]["float32"]
    m = c.model(ctx)
    pool = m.newPool(8, 1)
    t = dc.tokens(c.cfg, 37)
    got, want = m.captureLayers(t.size), []
    dc.run_steps(m, pool, [[("a", t)]])
    N.forward(c.cfg, c.W, t, want)
    for g, w in zip(got, want):
        assert np.abs(g - w).max() < 2e-5 * np.abs(w).max()
    pool.close(), m.close()


# ---- each mechanism alone ----------------------------------------------------------------------------------
def _alone(ctx, layer, dtype, sizes=(200, 1, 2, 40, 7, 50), width=64, edit=None, seed=3, tol=0.03, skip=None):
    """One layer on the embeddings of random tokens, in portions; skip(x, L): positions that are not compared."""
    cfg = nc.config([layer], width=width)
    W = nc.weights(cfg, seed)
    if edit:
        edit(W)
    W = {k: dc.bf16(v) for k, v in W.items()}
    m = D.DecoderModel(ctx, registry.describe(cfg, lambda k: W[k].shape), dtype, max(sizes))
    m.loadTensors(W.__getitem__)
    n = sum(sizes)
    pool = m.newPool(-(-n // 16), 1)
    t, want, got = dc.tokens(cfg, n, 5), [], []
    seq = pool.seq_alloc()
    for part in dc.cut(t, list(sizes)):
        cap = m.captureLayers(len(part))
        m.step(pool, [seq], [part], want_logits=False)
        got.append(cap[0])
    N.forward(cfg, W, t, want)
    d = np.abs(np.concatenate(got) - want[0])
    if dtype == "float32":
        assert d.max() < 3e-5 * np.abs(want[0]).max()
    else:
        d = np.sqrt((d * d).mean(-1)) / np.sqrt((want[0] ** 2).mean(-1))
        if skip is not None:
            keep = ~skip(cfg, W, t)
            assert keep.mean() > 0.6
            d = d[keep]
        assert d.max() < tol, (d.max(), int(d.argmax()))
    pool.close(), m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [dict(), dict(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2), dict(heads=33, kv_heads=1, dim=16, vdim=24),
                                dict(dim=128, vdim=128, rot_dims=128), dict(dim=90, vdim=33, rot_dims=50), dict(dim=60, vdim=30, rot_dims=28),
                                dict(heads=2, dim=130, vdim=190, rot_dims=20), dict(dim=31, vdim=60, rot_dims=6)])
def test_gated_attention_alone(ctx, kw, dtype):
    _alone(ctx, nc.att(mlp=None, **kw), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [dict(), dict(heads=1, kv_heads=1, dim=6, vdim=16), dict(heads=18, kv_heads=1, dim=16, vdim=32), dict(dim=64, vdim=128, yarn=None),
                                dict(dim=44, vdim=90, rot_dims=44), dict(heads=9, kv_heads=3, dim=128, vdim=256), dict(dim=90, vdim=180, rot_dims=10),
                                dict(dim=128, vdim=100, rot_dims=62), dict(dim=24, vdim=50, at=0.9)])
def test_differential_attention_alone(ctx, kw, dtype):
    _alone(ctx, nc.diff(mlp=None, **kw), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_head_norms_and_rotations_stand_out(ctx, dtype):
    """Norm weights that differ by orders between dimensions (a pair exchanged or a weight misplaced shows), heads that are tiny."""
    for layer, names in ((nc.att(mlp=None, dim=24, rot_dims=10), ("q.b", "k.b")), (nc.diff(mlp=None, dim=24, rot_dims=10), ())):
        def edit(W, names=names):
            for n in ("q.norm", "k.norm"):
                W["l0.mix." + n] = np.exp(np.linspace(-2, 1.2, 24))[np.random.default_rng(len(n) + ord(n[0])).permutation(24)]
            for n in ("q", "k"):
                W["l0.mix." + n] = W["l0.mix." + n] * 2e-3  # the norm's eps matters
            for n in names:
                W["l0.mix." + n] = W["l0.mix." + n] * 2e-3
        _alone(ctx, layer, dtype, edit=edit, tol=0.05)


def _near_choices(cfg, W, t):
    L = R.sub({k: np.asarray(v, np.float64) for k, v in W.items()}, "l0.")
    mixer = {"attention": N.gated_attention, "attention_2": N.differential_attention}[cfg["layers"][0]["type"]]
    x = W["embed"][t].astype(np.float64) * cfg["embedding"]["scale"]
    e = cfg["norm"]["eps"]
    x = N.rms_norm(cfg["postln_alpha"] * x + mixer(x, R.sub(L, "mix."), cfg["layers"][0]["mixer"], e), L["norm1"], e)
    z = R.linear(x, L["mlp.router"])
    return np.array([N.route_margin(v, L["mlp.correction"], cfg["layers"][0]["mlp"]["router"]) < min(0.004, 0.04 / v.size) for v in z])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", [nc.moe(), nc.moe(1, 0, 1, 1, 1), nc.moe(4, 0, 4, 1, 1, ff=100), nc.moe(60, 4, 9, 8, 3, ff=40, shared=70), nc.moe(3, 5, 3, 2, 2, shared=0),
                                 nc.moe(2, 6, 4, 4, 3, ff=17, shared=9), nc.moe(300, 20, 2, 32, 5, ff=8, shared=8), nc.moe(4, 0, 2, 4, 3, ff=64), nc.dense(75), nc.dense(8)])
def test_feed_forward_alone(ctx, mlp, dtype):
    _alone(ctx, nc.att(mlp=mlp), dtype, sizes=(300, 1, 2, 3, 20, 24, 64, 128, 90), skip=_near_choices if mlp["kind"] == "moe" else None)
    _alone(ctx, nc.att(mlp=mlp), dtype, sizes=(130, 40, 1), width=77, skip=_near_choices if mlp["kind"] == "moe" else None)


@pytest.mark.parametrize("dtype", DTYPES)
def test_every_token_to_the_same_experts_and_to_identity_only(ctx, dtype):
    def same(W):
        W["l0.mlp.correction"] = np.array([-9, 3, -7, 5, -4, -6, -8, -3.0])
        W["l0.mlp.e1.up"] = W["l0.mlp.e1.up"] * 3

    def identity(W):
        W["l0.mlp.correction"] = np.array([-9, -9, -9, 2, 3, 4.0])
    _alone(ctx, nc.att(mlp=nc.moe(8, 0, 2, 1, 1)), dtype, sizes=(300, 33, 1), edit=same)
    _alone(ctx, nc.att(mlp=nc.moe(3, 3, 3, 2, 1)), dtype, sizes=(300, 33, 1), edit=identity)
    _alone(ctx, nc.att(mlp=nc.moe(3, 3, 3, 1, 1, shared=0)), dtype, sizes=(300, 33, 1), edit=identity)


# ---- how a sequence is cut must not matter -------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[1], [2], [3, 2, 7], [16], [17], [64, 1, 1, 2], [150, 1]])
def test_portions_equal_the_whole(ctx, cases, sizes, dtype):
    for name in ("order", "ragged_sizes"):
        c = cases[name][dtype]
        m = c.model(ctx, dtype)
        pool = m.newPool(24, 2)
        t = dc.tokens(c.cfg, 190, 3)
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), dtype)
        pool.close(), m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(ctx, cases, dtype):
    c = cases["both"][dtype]
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
    c = cases[name][dtype]
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
    c = cases["both"]["bfloat16"]
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
    """Steps of single tokens at every length of a page, as many sequences as take another split of the keys and other tiles of
    the experts' rows, replayed graphs."""
    c = cases["large_heads"]["bfloat16"]
    m = c.model(ctx, "bfloat16")
    for n in (1, 5, 40, 140):
        pool = m.newPool(n * 8, n)
        toks = [dc.tokens(c.cfg, 60 + 3 * (i % 17), 500 + i) for i in range(n)]
        seqs = [pool.seq_alloc() for _ in range(n)]
        for i in range(0, n, 4):
            m.step(pool, seqs[i:i + 4], [t[:-20] for t in toks[i:i + 4]], want_logits=False)
        for j in range(20):
            if j % 5 == 4:
                logits, _ = m.step(pool, seqs, [t[len(t) - 20 + j:][:1] for t in toks], np.arange(n))
                for i in range(0, min(n, 40), 7):
                    _close(logits[i:i + 1], c.ref(toks[i])[len(toks[i]) - 20 + j:][:1], "bfloat16", 0.08)
            else:
                lens = [len(t) - 20 + j for t in toks]
                m.forwardDecodeBatch(pool, seqs, [t[k] for t, k in zip(toks, lens)], lens, want_logits=False)
        pool.close()
    m.close()


# ---- far keys, first tokens ------------------------------------------------------------------------------------
def _needle(cfg, needle=1, query=2):
    """Weights with which a query of the `query` token falls on keys of the `needle` token alone: its projection is that of the
    needle's key, the norms make equal heads score high (and keep the rotated dimensions small)."""
    def edit(W):
        n, q = (W["embed"][i].astype(np.float64) for i in (needle, query))
        for i, e in enumerate(cfg["layers"]):
            p, m = f"l{i}.mix.", e["mixer"]
            maps = 2 if e["type"] == "attention_2" else 1
            k = W[p + "k"].reshape(m["kv_heads"], maps * m["dim"], -1)
            k = np.repeat(k, m["heads"] // m["kv_heads"], 0).reshape(-1, cfg["width"])
            W[p + "q"] = k + np.outer(k @ (n - q), q) / (q @ q)
            if maps == 1:
                W[p + "q.b"], W[p + "k.b"] = W[p + "q.b"] * 0, W[p + "k.b"] * 0
            for x in ("q.norm", "k.norm"):
                W[p + x] = np.where(np.arange(m["dim"]) < m["rot"]["dims"], 0.4, 2.2)
    return edit


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [nc.att(dim=24, vdim=32, rot_dims=4, base=1e5, scale=0.35, mlp=None),
                                   nc.diff(dim=24, vdim=32, rot_dims=4, base=1e5, scale=0.35, mlp=None)], ids=["gated", "differential"])
def test_one_far_key_among_hundreds(ctx, layer, dtype):
    """A key at a sequence's start, a page's edges or just before the query decides the query's output."""
    cfg = nc.config([layer], alpha=0.5)
    c = nc.Case(cfg, seed=6, edit=_needle(cfg))
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
            _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], want, dtype, None if dtype == "float32" else 0.1)
    pool.close(), m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(ctx, cases, dtype):
    """Sequences of one to five tokens, whole and token by token, in slots that longer ones have left."""
    c = cases["both"][dtype]
    m = c.model(ctx, dtype)
    pool = m.newPool(6, 1)
    dc.run_steps(m, pool, [[("x", dc.tokens(c.cfg, 90, 9))]])
    for n in range(1, 6):
        t = dc.tokens(c.cfg, n, 70 + n)
        for sizes in ([n], [1], [2, 1]):
            _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), dtype)
    pool.close(), m.close()


def test_positions_far_from_the_start(ctx):
    """Rotations of large positions, plain and scaled, against float64 angles."""
    cfg = nc.config([nc.att(base=50.0, heads=2, mlp=None), nc.diff(base=60.0, heads=2, kv_heads=1, mlp=None)])
    c = nc.Case(cfg, seed=2)
    m = c.model(ctx)
    pool = m.newPool(160, 1)
    t = dc.tokens(cfg, 2000, 6)
    _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, [500])])["a"], c.ref(t), "float32")
    pool.close(), m.close()


# ---- scheduler, generation -----------------------------------------------------------------------------------
def test_greedy_generation_equals_the_oracle(ctx, cases):
    c = cases["ragged_sizes"]["float32"]
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
    c = cases["both"][dtype]
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
            lg = N.forward(c.cfg, c.W, np.concatenate([p, got]))  # every pick is near the oracle's best
            for j, tok in enumerate(got):
                row = lg[len(p) - 1 + j]
                assert row.max() - row[tok] < 0.25 * row.std()
    batch.close(), pool.close(), m.close()


def test_misfits_are_refused(ctx):
    def build(layers, **kw):
        c = nc.Case(nc.config(layers, **kw))
        c.model(ctx).close()
    for mlp in (nc.moe(7, 0, 3, 2, 1), nc.moe(6, 0, 4, 2, 1), nc.moe(6, 0, 2, 2, 3)):  # unequal groups, too few to choose from, too many kept
        with pytest.raises((ValueError, IndexError)):
            build([nc.att(mlp=mlp)])
    with pytest.raises(ValueError):  # more than the head turns
        build([nc.att(dim=8, rot_dims=10)])


def test_command_lines(ctx, cases, tmp_path):
    from jgpt_b200 import safetensors

    c = cases["both"]["float32"]
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
