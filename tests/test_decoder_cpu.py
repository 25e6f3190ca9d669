"""Layered decoders, host side: registry, weight files, ABI structures, trace handling, and the oracle's own invariants."""
import ctypes as C
import io
import json
import os
import re

import numpy as np
import pytest

import decoder_cases as dc
from jgpt_b200 import decoder as D
from jgpt_b200 import registry, safetensors, trace
from oracle import hybrid_ref as R

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---- registry and files --------------------------------------------------------------------------------
def test_registry_reads_every_size_from_config_and_shapes():
    cfg = dc.config([dc.delta(heads=6, kv_heads=3, conv=5, ff=36), dc.par(left=dc.attn(size=19, scale=0.21), right=dc.gla(tau=3.5), ff=0)], width=52)
    W = dc.weights(cfg, rank_a=7, rank_g=9)
    d = registry.describe(cfg, lambda n: W[n].shape)
    assert (d.vocab, d.width, d.max_positions, d.eps, d.embed_scale, d.logit_scale) == (101, 52, 640, 2e-5, 2.5, 0.3)
    a, b = d.layers
    assert a.ff == 36 and b.ff == 0 and len(a.branches) == 1 and len(b.branches) == 2
    m = a.branches[0]
    assert (m.kind, m.heads, m.kv_heads, m.dim, m.vdim, m.taps, m.rank_a, m.rank_g) == (D.MIX_DELTA, 6, 3, 24, 20, 5, 7, 9)
    at, gl = b.branches
    assert (at.kind, at.chunk, at.score_scale, at.out_scale, at.gate) == (D.MIX_ATTENTION, 19, 0.21, 0.7, True)
    assert (gl.kind, gl.tau, gl.out_scale, gl.rank_a) == (D.MIX_GLA, 3.5, 1.3, 7)
    assert {n for *_, n in d.all_tensors()} == set(W)  # nothing is left over, nothing is made up


def test_unknown_designs_and_parts_are_refused():
    cfg = dc.config([dc.par()])
    shape = lambda n: dc.weights(cfg)[n].shape  # noqa: E731
    with pytest.raises(ValueError, match="not registered"):
        registry.describe({**cfg, "architecture": "Nameless"}, shape)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "mystery"
    with pytest.raises(ValueError, match="mixer type"):
        registry.describe(bad, shape)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError, match="feed-forward"):
        registry.describe(bad, shape)


def test_safetensors_round_trip_and_errors(tmp_path):
    x = {"a": dc.bf16(np.random.default_rng(0).standard_normal((3, 5))), "b": np.arange(4, dtype=np.float32)}
    path = tmp_path / "w.safetensors"
    safetensors.write_bf16(path, x)
    f = safetensors.SafetensorsFile(path)
    assert set(f.names()) == {"a", "b"} and f.shape("a") == (3, 5) and "c" not in f
    for k in x:
        assert np.array_equal(f.get(k), x[k])
    with pytest.raises(KeyError):
        f.get("c")
    head = json.dumps({"i": {"dtype": "I32", "shape": [2], "data_offsets": [0, 8]}, "z": {"dtype": "F8_X", "shape": [1], "data_offsets": [8, 9]}}).encode()
    p2 = tmp_path / "i.safetensors"
    p2.write_bytes(len(head).to_bytes(8, "little") + head + np.array([7, -2], np.int32).tobytes() + b"\0")
    g = safetensors.SafetensorsFile(p2)
    assert g.get("i").tolist() == [7, -2]
    with pytest.raises(ValueError, match="dtype"):
        g.get("z")


def test_bf16_rounds_to_nearest_even():
    one = np.float32(1.0)
    ulp = np.float32(2.0 ** -7)
    assert dc.bf16([one + ulp / 2])[0] == one and dc.bf16([one + ulp * 1.5])[0] == one + 2 * ulp
    assert dc.bf16([one + ulp * 0.51])[0] == one + ulp


def test_abi_structures_match_the_header():
    src = open(os.path.join(ROOT, "include", "jgpt_b200.h")).read()
    src = re.sub(r"/\*.*?\*/", "", src, flags=re.S)

    def fields(name):
        body = re.search(r"typedef struct \{([^{}]*)\} %s;" % name, src).group(1)
        out = []
        for t, names in re.findall(r"(int32_t|float|double|jgpt_\w+_spec)\s+([^;]+);", body):
            out += [(n.strip().split("[")[0], t) for n in names.split(",")]
        return out

    ct = {C.c_int32: "int32_t", C.c_float: "float", C.c_double: "double", D._MixerSpec * D.MAX_BRANCHES: "jgpt_mixer_spec", D._MoeSpec: "jgpt_moe_spec"}
    for name, cls in (("jgpt_mixer_spec", D._MixerSpec), ("jgpt_moe_spec", D._MoeSpec), ("jgpt_layer_spec", D._LayerSpec), ("jgpt_decoder_spec", D._DecoderSpec)):
        assert fields(name) == [(n, ct[t]) for n, t in cls._fields_], name
    roles = re.search(r"JGPT_W_EMBED = 0.*?\};", src, re.S).group(0)
    at, value = -1, {}
    for n, v in re.findall(r"(JGPT_W_\w+)(?:\s*=\s*(\d+))?", roles):
        at = int(v) if v else at + 1
        value[n] = at
    for n, v in value.items():
        assert getattr(D, n.replace("JGPT_", "")) == v, n


# ---- trace -----------------------------------------------------------------------------------------------
def test_steps_longer_than_the_workspace_are_cut():
    assert trace.split_step([3, 1], 8) == [[(0, 0, 3), (1, 0, 1)]]
    assert trace.split_step([5, 4], 4) == [[(0, 0, 4)], [(0, 4, 1), (1, 0, 3)], [(1, 3, 1)]]
    assert trace.split_step([4], 4) == [[(0, 0, 4)]]


def test_trace_replay_orders_logits_and_gives_slots_back(tmp_path):
    class Pool:
        def __init__(self, n):
            self.free, self.log = list(range(n))[::-1], []

        def seq_alloc(self):
            return self.free.pop()

        def seq_free(self, s):
            self.free.append(s)

        def close(self):
            self.log.append("closed")

    class Model:
        maxRows = 4

        def newPool(self, blocks, seqs):
            assert blocks == 8 and seqs == 4  # 128 tokens in blocks of 16
            self.pool = Pool(seqs)
            return self.pool

        def step(self, pool, seqs, toks, want, want_logits):
            flat = np.concatenate(toks)
            assert flat.size <= self.maxRows
            return np.array([[flat[w], 0.5] for w in want], np.float32), None

    m, out = Model(), io.StringIO()
    lines = [json.dumps(s) for s in (
        {"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7, 8, 9], "want": [4, 0]}, {"id": "b", "tokens": [3], "want": [0]}], "end": ["b"]},
        {"step": 1, "entries": [{"id": "c", "tokens": [1, 2], "want": []}], "end": ["a", "c"]})]
    trace.replay(m, lines, out, str(tmp_path), 128)
    assert out.getvalue().splitlines() == ["done 0", "done 1"]
    got = np.fromfile(tmp_path / "0.f32", np.float32).reshape(-1, 2)
    assert got[:, 0].tolist() == [9, 5, 3]  # the order of the entries and of 'want'
    assert not (tmp_path / "1.f32").exists() and sorted(m.pool.free) == [0, 1, 2, 3]


# ---- the oracle's own invariants ---------------------------------------------------------------------------
def test_chunk_rule():
    v = R.chunk_visible(10, 4)
    assert v[3].tolist() == [True] * 4 + [False] * 6  # last of its chunk
    assert v[4].tolist() == [False] * 4 + [True] + [False] * 5  # first of the next
    assert R.chunk_visible(5, 0).sum() == 15 and R.chunk_visible(5, 1).sum() == 5


def test_gla_scan_is_the_decayed_sum():
    rng = np.random.default_rng(0)
    q, k, a = (rng.random((6, 2, 3)) for _ in range(3))
    v = rng.random((6, 2, 4))
    o = R.gla_scan(q, k, v, a)
    for t in range(6):
        want = sum(np.einsum("hk,hv->hv", q[t] * k[j] * np.prod(a[j + 1:t + 1], 0), v[j]) for j in range(t + 1))
        assert np.allclose(o[t], want)


def test_delta_rule_writes_what_it_should_read():
    """With beta 1 and no decay, reading with the key that was just written gives the value back."""
    rng = np.random.default_rng(1)
    k = R.unit(rng.standard_normal((5, 1, 8)) * 1e3)
    v = rng.standard_normal((5, 1, 4))
    o = R.delta_scan(k, k, v, np.ones_like(k), np.ones((5, 1)))
    assert np.allclose(o, v, atol=1e-6)
    half = R.delta_scan(k, k, v, np.ones_like(k), np.full((5, 1), 0.5))
    assert np.allclose(half[0], 0.5 * v[0], atol=1e-6)


def test_short_conv_last_column_is_the_current_token():
    x = np.array([[1.0], [2.0], [4.0]])
    assert R.short_conv(x, [[0.0, 0.0, 1.0]]).ravel().tolist() == [1, 2, 4]
    assert R.short_conv(x, [[1.0, 0.0, 0.0]]).ravel().tolist() == [0, 0, 1]
    assert R.short_conv(x, [[3.0]]).ravel().tolist() == [3, 6, 12]


def test_oracle_is_causal_and_chunked():
    cfg = dc.config([dc.delta(), dc.par()], positions=40)
    W = dc.weights(cfg)
    a = dc.tokens(cfg, 30)
    b = a.copy()
    b[20] = b[20] % (cfg["vocab"] - 1) + 1
    x, y = R.forward(cfg, W, a), R.forward(cfg, W, b)
    assert np.allclose(x[:20], y[:20]) and not np.allclose(x[20], y[20])
