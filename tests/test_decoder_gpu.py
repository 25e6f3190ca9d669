"""Layered decoders on the GPU against the plain oracle (oracle/hybrid_ref.py): mechanisms alone and together, prompts,
decoding, portions, mixed batches, blocks and slots used again, chunk edges, the scheduler and generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import decoder_cases as dc
from jgpt_b200 import ContinuousBatcher, PoolExhausted
from jgpt_b200 import decoder as D
from oracle import hybrid_ref as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL, BF16_TOL = 3e-5, 0.05

CASES = {
    "both": dc.config([dc.delta(), dc.par()]),
    "order": dc.config([dc.par(ff=0), dc.par(ls=1.9, rs=0.2), dc.delta(ff=33), dc.delta(heads=3, kv_heads=3, conv=2)], width=96, vocab=128),
    "ragged_sizes": dc.config([dc.par(left=dc.attn(heads=6, kv_heads=3, dim=20, vdim=28, size=17), right=dc.gla(heads=5, dim=12, vdim=36, tau=1.0), ff=50),
                               dc.delta(heads=6, kv_heads=2, dim=40, vdim=12, conv=5, ff=70)], width=76, vocab=93),
    "one_tap_one_head": dc.config([dc.delta(heads=1, kv_heads=1, conv=1), dc.par(left=dc.attn(heads=1, kv_heads=1, size=1), right=dc.gla(heads=1))], width=44),
    "large_heads": dc.config([dc.par(left=dc.attn(heads=2, kv_heads=1, dim=128, vdim=96, size=50), right=dc.gla(heads=2, dim=128, vdim=64)),
                              dc.delta(heads=2, kv_heads=1, dim=96, vdim=128, conv=3), dc.delta(heads=1, kv_heads=1, dim=200, vdim=176, conv=3),
                              dc.par(left=dc.attn(heads=10, kv_heads=1, dim=32, vdim=160, size=40), right=dc.gla(heads=1, dim=256, vdim=256))], width=128),
    "wide_groups": dc.config([dc.par(left=dc.attn(heads=24, kv_heads=1, dim=16, vdim=16, size=37)), dc.par(left=dc.attn(heads=12, kv_heads=4, size=150))]),
}


@pytest.fixture(scope="module")
def cases():
    return {k: dc.Case(c, seed=i) for i, (k, c) in enumerate(CASES.items())}


def _close(got, want, dtype):
    e = dc.error(got, want)
    assert np.isfinite(e).all() and e.max() < (F32_TOL if dtype == "float32" else BF16_TOL), (dtype, e.max(), int(e.argmax()))


# ---- the model against the oracle --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CASES))
def test_prompt_matches_the_oracle(ctx, cases, name, dtype):
    c = cases[name]
    m = c.model(ctx, dtype)
    pool = m.newPool(60, 3)
    for n in (1, 2, 131, 333):  # below and above the rows from which the tcgen05 products run
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
    R.forward(c.cfg, c.W, t, want)
    for g, w in zip(got, want):
        assert np.abs(g - w).max() < 2e-5 * np.abs(w).max()
    pool.close(), m.close()


# ---- each mechanism alone ----------------------------------------------------------------------------------
def _alone(ctx, mixer_spec, weights, apply, dtype, n=70, width=64):
    """A one-layer model x + mixer(LN(x)) built without the registry; compares the residual after the layer."""
    rng = np.random.default_rng(5)
    top = {"e": dc.bf16(rng.standard_normal((50, width))), "p": dc.bf16(rng.standard_normal((128, width))), "one": np.ones(width, np.float32),
           "zero": np.zeros(width, np.float32)}
    cfg = D.DecoderConfig(50, width, 128, 1e-5, [D.Layer([mixer_spec], 0, {D.W_NORM1: "one", D.W_NORM1_B: "zero"})],
                          tensors={D.W_EMBED: "e", D.W_POS: "p", D.W_FINAL_NORM: "one", D.W_FINAL_NORM_B: "zero"})
    m = D.DecoderModel(ctx, cfg, dtype, 128)
    m.loadTensors(lambda k: top[k] if k in top else weights[k])
    pool = m.newPool(8, 1)
    t = rng.integers(0, 50, n).astype(np.int32)
    cap = m.captureLayers(n)
    m.step(pool, [pool.seq_alloc()], [t], want_logits=False)
    x = top["e"][t].astype(np.float64) + top["p"][:n]
    want = apply(R.layer_norm(x, 1.0, 0.0, 1e-5)) * mixer_spec.out_scale
    got = cap[0] - x
    assert np.abs(got - want).max() < (1e-5 if dtype == "float32" else 0.03) * np.abs(want).max()
    pool.close(), m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk,gate", [(0, True), (13, True), (32, False), (200, True)])
def test_attention_alone(ctx, chunk, gate, dtype):
    a = dc.attn(heads=6, kv_heads=2, dim=24, vdim=40, size=chunk)
    cfg = dc.config([dc.par(left=a)], width=64)
    W = R.sub({k: v for k, v in dc.weights(cfg).items()}, "l0.mix.left.")
    names = {D.W_Q: "q", D.W_K: "k", D.W_V: "v", D.W_O: "o"}
    if gate:
        names[D.W_G] = "g"
    spec = D.Mixer(D.MIX_ATTENTION, 6, 2, 24, 40, chunk=chunk, gate=gate, score_scale=0.4, out_scale=0.6, tensors=names)
    F = {k: np.asarray(v, np.float64) for k, v in W.items()}

    def apply(h):
        if gate:
            return R.gated_chunk_attention(h, F, {**a, "scale": 0.4})
        q, k, v = R.linear(h, F["q"]).reshape(-1, 6, 24), R.linear(h, F["k"]).reshape(-1, 2, 24), R.linear(h, F["v"]).reshape(-1, 2, 40)
        return R.linear(R.attention(q, k, v, 0.4, chunk).reshape(len(h), -1), F["o"])
    _alone(ctx, spec, W, apply, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tau", [0.5, 16.0])
def test_gated_linear_attention_alone(ctx, tau, dtype):
    g = dc.gla(heads=3, dim=48, vdim=40, tau=tau)
    W = R.sub(dc.weights(dc.config([dc.par(right=g)], width=64)), "l0.mix.right.")
    spec = D.Mixer(D.MIX_GLA, 3, 3, 48, 40, rank_a=6, tau=tau, out_scale=1.7,
                   tensors={D.W_Q: "q", D.W_K: "k", D.W_V: "v", D.W_G: "g", D.W_O: "o", D.W_A1: "a1", D.W_A2: "a2", D.W_DECAY_BIAS: "a2.b",
                            D.W_HEAD_NORM: "norm"})
    F = {k: np.asarray(v, np.float64) for k, v in W.items()}
    _alone(ctx, spec, W, lambda h: R.gated_linear_attention(h, F, g, 1e-5), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("taps,heads,kv", [(1, 2, 2), (3, 4, 2), (8, 4, 1)])
def test_delta_rule_alone(ctx, taps, heads, kv, dtype):
    d = dc.delta(heads=heads, kv_heads=kv, dim=40, vdim=24, conv=taps)
    W = R.sub(dc.weights(dc.config([d], width=64)), "l0.mix.")
    spec = D.Mixer(D.MIX_DELTA, heads, kv, 40, 24, taps=taps, rank_a=6, rank_g=10, out_scale=0.9,
                   tensors={D.W_Q: "q", D.W_K: "k", D.W_V: "v", D.W_O: "o", D.W_B: "b", D.W_A1: "a1", D.W_A2: "a2", D.W_DECAY_BIAS: "dt_bias",
                            D.W_A_LOG: "A_log", D.W_G1: "g1", D.W_G2: "g2", D.W_HEAD_NORM: "norm", D.W_CONV_Q: "q.conv", D.W_CONV_K: "k.conv",
                            D.W_CONV_V: "v.conv"})
    F = {k: np.asarray(v, np.float64) for k, v in W.items()}
    _alone(ctx, spec, W, lambda h: R.channel_delta(h, F, d["mixer"], 1e-5), dtype)


# ---- how a sequence is cut must not matter -------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [[1], [2], [3, 2, 7], [16], [17], [64, 1, 1, 2], [150, 1]])
def test_portions_equal_the_whole(ctx, cases, sizes, dtype):
    for name in ("order", "ragged_sizes"):
        c = cases[name]
        m = c.model(ctx, dtype)
        pool = m.newPool(24, 2)
        t = dc.tokens(c.cfg, 190, 3)
        got = dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"]
        _close(got, c.ref(t), dtype)
        pool.close(), m.close()


@pytest.mark.parametrize("name", list(CASES))
def test_chunked_recurrences_at_full_precision(ctx, cases, name, monkeypatch):
    """The chunked form of the recurrences (tensor cores, three TF32 products) on fp32 activations: as close to the oracle as
    the token-by-token form, for whole prompts, for portions around the length from which it is used, and beside short ones."""
    monkeypatch.setenv("JGPT_B200_REC_CHUNK_EXACT", "1")
    monkeypatch.setenv("JGPT_B200_REC_CHUNK_MIN", "6")
    c = cases[name]
    m = c.model(ctx, "float32")
    pool = m.newPool(60, 3)
    for sizes in ([320], [6], [5, 7, 1, 40, 2, 16, 17, 33], [161, 1, 158]):
        t = dc.tokens(c.cfg, 320, 17)
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), "float32")
    toks = {f"r{i}": dc.tokens(c.cfg, L, 50 + i) for i, L in enumerate([1, 150, 33, 64, 17, 2])}
    got = dc.run_steps(m, pool, dc.mixed_plan(toks, 3))
    for r, t in toks.items():
        _close(got[r], c.ref(t), "float32")
    pool.close(), m.close()


def test_chunked_recurrences_with_decays_that_vanish(ctx, monkeypatch):
    """Channels that forget everything from one token to the next, beside channels that forget nothing."""
    monkeypatch.setenv("JGPT_B200_REC_CHUNK_EXACT", "1")
    cfg = dc.config([dc.delta(heads=2, kv_heads=2, dim=32, vdim=16), dc.par(right=dc.gla(heads=2, dim=32, vdim=16, tau=0.1))])

    def edit(W):
        W["l0.mix.A_log"] = np.array([4.0, -8.0])
        W["l0.mix.dt_bias"] = W["l0.mix.dt_bias"] * 4
        W["l1.mix.right.a2.b"] = W["l1.mix.right.a2.b"] * 10 - 20
    c = dc.Case(cfg, seed=4, edit=edit)
    t = dc.tokens(cfg, 200, 1)
    for dtype in ("float32", "bfloat16"):
        m = c.model(ctx, dtype)
        pool = m.newPool(16, 1)
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, [100, 1, 99])])["a"], c.ref(t), dtype)
        pool.close(), m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(ctx, cases, dtype):
    c = cases["both"]
    m = c.model(ctx, dtype)
    pool = m.newPool(40, 1)
    t = dc.tokens(c.cfg, 500, 4)
    got = dc.run_steps(m, pool, [[("a", t[:20])]] + [[("a", t[i:i + 1])] for i in range(20, 500)])["a"]
    _close(got, c.ref(t), dtype)
    pool.close(), m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["order", "ragged_sizes", "wide_groups"])
def test_mixed_batches_with_blocks_and_slots_used_again(ctx, cases, name, dtype):
    """Nine requests through three slots and a pool that holds far fewer blocks than they need together, on storage that
    starts as NaN patterns: what a request reads, it or nobody has written."""
    c = cases[name]
    m = c.model(ctx, dtype)
    pool = m.newPool(40, 3)
    p, n = pool.storage()
    from jgpt_b200 import binding as B
    B.check(m._lib.jgpt_dev_memset(ctx.handle, p, 0xFF, n))
    toks = {f"r{i}": dc.tokens(c.cfg, L, 50 + i) for i, L in enumerate([1, 150, 33, 200, 64, 17, 2, 180, 90])}
    got = dc.run_steps(m, pool, dc.mixed_plan(toks, 7))
    for r, t in toks.items():
        _close(got[r], c.ref(t), dtype)
    assert pool.free_blocks() == 40
    pool.close(), m.close()


def test_batch_of_unequal_requests_equals_each_alone(ctx, cases):
    c = cases["both"]
    m = c.model(ctx, "bfloat16")
    pool = m.newPool(80, 6)
    toks = {f"r{i}": dc.tokens(c.cfg, L, 80 + i) for i, L in enumerate([5, 1, 64, 130, 2, 17])}
    together = dc.run_steps(m, pool, [list(toks.items())])
    for r, t in toks.items():
        alone = dc.run_steps(m, pool, [[(r, t)]])[r]
        assert dc.error(together[r], alone.astype(np.float64)).max() < 0.03
        _close(together[r], c.ref(t), "bfloat16")
    pool.close(), m.close()


# ---- edges -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("size", [1, 15, 16, 17, 31, 33, 64, 100])
def test_chunk_edges_stand_out(ctx, size):
    """Scores are scaled up so that a query's weight sits on few keys: a key too many or too few at a chunk's or a block's
    edge changes the logits of that position, shown on the oracle itself with the chunk one token longer."""
    left = dc.attn(heads=4, kv_heads=2, dim=16, vdim=16, size=size, scale=2.0)
    cfg = dc.config([dc.par(left=left, ls=2.0, rs=0.1, ff=0)], positions=256)
    c = dc.Case(cfg, seed=size)
    t = dc.tokens(cfg, 210, size)
    want = c.ref(t)
    wrong = json.loads(json.dumps(cfg))
    wrong["layers"][0]["mixer"]["left"]["mask"]["size"] = size + 1
    assert dc.error(c.ref(t, wrong), want).max() > 0.3
    for dtype in ("float32", "bfloat16"):
        m = c.model(ctx, dtype)
        pool = m.newPool(14, 1)
        for sizes in ([210], [37, 1, 1, 30, 2], [205, 1], [1]):
            e = dc.error(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], want)
            assert e.max() < (F32_TOL if dtype == "float32" else 0.1), (dtype, sizes, e.max(), int(e.argmax()))
        pool.close(), m.close()


def test_a_far_key_is_found_through_the_recurrent_state(ctx):
    """Slow decays and one key direction: a value written in the first tokens still shows hundreds of tokens later."""
    cfg = dc.config([dc.delta(heads=2, kv_heads=1, dim=16, vdim=16, conv=3), dc.par(right=dc.gla(heads=2, dim=16, vdim=16, tau=64.0), ls=0.1, rs=2.0)])

    def slow(W):
        W["l0.mix.A_log"] = W["l0.mix.A_log"] * 0 - 8.0
        W["l1.mix.right.a2.b"] = W["l1.mix.right.a2.b"] * 0 + 6.0
    c = dc.Case(cfg, seed=3, edit=slow)
    t = dc.tokens(cfg, 600, 1)
    u = t.copy()
    u[3] = u[3] % (cfg["vocab"] - 1) + 1
    assert dc.error(c.ref(u)[-1:], c.ref(t)[-1:]).max() > 20 * F32_TOL  # the early token shows at the end
    m = c.model(ctx, "float32")
    pool = m.newPool(40, 1)
    for toks in (t, u):
        for sizes in ([600 - 88, 60, 1], [7, 2, 93]):
            plan = [[("a", p)] for p in dc.cut(toks, sizes)]
            if max(len(p[0][1]) for p in plan) <= m.maxRows:
                _close(dc.run_steps(m, pool, plan)["a"], c.ref(toks), "float32")
    pool.close(), m.close()


def test_first_tokens_and_convolution_history(ctx):
    """The convolution's window reaches before the start, across portions shorter than itself, and not into a slot's
    previous owner."""
    cfg = dc.config([dc.delta(heads=4, kv_heads=2, conv=6), dc.delta(heads=2, kv_heads=2, conv=4)])
    c = dc.Case(cfg, seed=9)
    m = c.model(ctx)
    pool = m.newPool(8, 1)
    for i, sizes in enumerate(([1], [2], [3], [1, 2, 4, 2, 1], [5], [40])):
        t = dc.tokens(cfg, 40, i)
        _close(dc.run_steps(m, pool, [[("a", p)] for p in dc.cut(t, sizes)])["a"], c.ref(t), "float32")
    pool.close(), m.close()


# ---- scheduler, generation, sampling -------------------------------------------------------------------------
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_continuous_batching(ctx, cases, dtype):
    """Requests through the framework's scheduler: prompts in portions beside decoded tokens, finished sequences evicted for
    room.  Each stream equals the one the request has alone (fp32: the oracle's)."""
    c = cases["order"]
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
            lg = R.forward(c.cfg, c.W, np.concatenate([p, got]))  # every pick is near the oracle's best
            for j, tok in enumerate(got):
                row = lg[len(p) - 1 + j]
                assert row.max() - row[tok] < 0.2 * row.std()
    assert {e[0] for e in batch.events()} == {1, 2, 3}
    batch.close(), pool.close(), m.close()


def test_sampled_tokens_are_those_of_the_host_sampler(ctx, cases):
    import ctypes as C

    c = cases["both"]
    m = c.model(ctx, "float32")
    pool = m.newPool(8, 2)
    t = dc.tokens(c.cfg, 9, 1)
    u = np.float32([0.1, 0.77])
    seqs = [pool.seq_alloc(), pool.seq_alloc()]
    m.step(pool, seqs, [t, t[:4]], want_logits=False)
    got = m.forwardDecodeSampleBatch(pool, seqs, [5, 6], [9, 4], 0.8, 7, u)
    for i, toks in enumerate(([*t, 5], [*t[:4], 6])):
        lg = np.ascontiguousarray(c.ref(toks)[-1], np.float32)
        tok = C.c_int32()
        m._lib.jgpt_sample_next_token(lg.ctypes.data, lg.size, 0.8, 7, float(u[i]), C.byref(tok))
        assert tok.value == got[i]
    out = m.generateGpuKv(t, 6, temperature=0.7, topK=5, rng=np.random.default_rng(0))
    assert out.size == 15 and (out[:9] == t).all()
    pool.close(), m.close()


# ---- misuse --------------------------------------------------------------------------------------------------
def test_misuse_is_refused_and_changes_nothing(ctx, cases):
    c = cases["both"]
    m = c.model(ctx, "float32", max_rows=64)
    pool = m.newPool(3, 2)
    a, b = pool.seq_alloc(), pool.seq_alloc()
    t = dc.tokens(c.cfg, 30, 0)
    m.step(pool, [a], [t], want_logits=False)
    with pytest.raises(PoolExhausted):  # two blocks each: neither keeps what it was given
        m.step(pool, [a, b], [t[:10], t[:20]], want_logits=False)
    assert pool.free_blocks() == 1 and pool.length(a) == 30 and pool.length(b) == 0
    for seqs, toks, err in (([a, a], [t[:1], t[:1]], ValueError), ([7], [t[:1]], IndexError), ([b], [[c.cfg["vocab"]]], IndexError),
                            ([b], [np.zeros(65, np.int32)], ValueError)):
        with pytest.raises(err):
            m.step(pool, seqs, toks, want_logits=False)
    with pytest.raises(RuntimeError):
        pool.set_length(a, 7)  # recurrent state cannot go back
    with pytest.raises(RuntimeError):
        m.forwardDecodeBatch(pool, [a], [1], [3])
    lg, _ = m.step(pool, [a], [t[:2]], [1])
    _close(lg, c.ref(np.concatenate([t, t[:2]]))[-1:], "float32")
    short = D.DecoderModel(ctx, m.config, "float32", 16)
    with pytest.raises(RuntimeError, match="not set"):
        short.step(pool, [b], [t[:1]])
    with pytest.raises(ValueError):
        short.setTensor(0, 0, D.W_Q, np.zeros((3, 3)))
    short.close(), pool.close(), m.close()


# ---- command lines -------------------------------------------------------------------------------------------
def test_trace_run_and_generate_command_lines(ctx, cases, tmp_path):
    from jgpt_b200 import safetensors

    c = cases["both"]
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
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1"]
    want = c.ref(t)
    _close(np.fromfile(out / "0.f32", np.float32).reshape(2, -1), want[[32, 3]], "float32")
    _close(np.fromfile(out / "1.f32", np.float32).reshape(1, -1), want[[39]], "float32")
    r = subprocess.run([sys.executable, "-m", "jgpt_b200.generate", "--model", str(folder), "--dtype", "float32", "--prompt", ",".join(map(str, t[:5])),
                        "--prompt", ",".join(map(str, t[5:8])), "--max-new", "6"], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    lines = [json.loads(x) for x in r.stdout.splitlines() if x.startswith("{")]
    for line, p in zip(lines, (t[:5], t[5:8])):
        assert line["tokens"] == dc.greedy(c, p, 6)[0]
