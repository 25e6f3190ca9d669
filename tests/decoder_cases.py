"""Small layered decoders with random weights for the tests: configurations, weights (rounded to bfloat16, so that every
side computes with the same numbers), and the library's model built from them through the registry."""
from __future__ import annotations

import numpy as np

from jgpt_b200 import decoder as D
from jgpt_b200 import registry
from jgpt_b200.safetensors import bf16_to_f32, f32_to_bf16
from oracle import hybrid_ref as R


def attn(heads=4, kv_heads=2, dim=16, vdim=16, size=24, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale or dim ** -0.5}


def gla(heads=3, dim=16, vdim=24, tau=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def par(left=None, right=None, ls=0.7, rs=1.3, ff=48):
    return {"type": "parallel", "mixer": {"left": left or attn(), "right": right or gla(), "left_scale": ls, "right_scale": rs},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads=4, kv_heads=2, dim=24, vdim=20, conv=4, ff=0):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=80, vocab=101, positions=640, eps=2e-5, embed_scale=2.5, logit_scale=0.3):
    return {"architecture": "Somopel", "layers": layers, "width": width, "vocab": vocab, "max_positions": positions, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "logit_scale": logit_scale}


def bf16(x):
    return bf16_to_f32(f32_to_bf16(np.asarray(x, np.float32)))


def weights(cfg, seed=0, rank_a=6, rank_g=10):
    rng = np.random.default_rng(seed)
    W, w = {}, cfg["width"]

    def lin(name, out, inp, gain=1.0):
        W[name] = rng.standard_normal((out, inp)) * gain / np.sqrt(inp)

    def norm(name, n, bias=True):
        W[name] = 1 + 0.2 * rng.standard_normal(n)
        if bias:
            W[name + ".b"] = 0.2 * rng.standard_normal(n)

    W["embed"] = rng.standard_normal((cfg["vocab"], w))
    W["pos"] = rng.standard_normal((cfg["max_positions"], w))
    norm("embed.norm", w), norm("final.norm", w)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        norm(p + "norm1", w)
        if e["type"] == "parallel":
            a, b = m["left"], m["right"]
            q = p + "mix.left."
            lin(q + "q", a["heads"] * a["dim"], w), lin(q + "k", a["kv_heads"] * a["dim"], w), lin(q + "v", a["kv_heads"] * a["vdim"], w)
            lin(q + "g", a["heads"], w), lin(q + "o", w, a["heads"] * a["vdim"])
            q = p + "mix.right."
            lin(q + "q", b["heads"] * b["dim"], w), lin(q + "k", b["heads"] * b["dim"], w), lin(q + "v", b["heads"] * b["vdim"], w)
            lin(q + "g", b["heads"] * b["vdim"], w), lin(q + "o", w, b["heads"] * b["vdim"])
            lin(q + "a1", rank_a, w), lin(q + "a2", b["heads"] * b["dim"], rank_a, 2.0)
            W[q + "a2.b"] = rng.standard_normal(b["heads"] * b["dim"]) + 2
            norm(q + "norm", b["vdim"], bias=False)
        else:
            q, H, G, dk, dv = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for name, n in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                lin(q + name, n, w)
                W[q + name + ".conv"] = rng.standard_normal((n, m["conv"])) / np.sqrt(m["conv"]) + 0.2
            lin(q + "b", H, w, 2.0), lin(q + "o", w, H * dv)
            W[q + "A_log"] = rng.uniform(-3, 0.5, H)
            W[q + "dt_bias"] = rng.standard_normal(H * dk) - 1
            lin(q + "a1", rank_a, w), lin(q + "a2", H * dk, rank_a), lin(q + "g1", rank_g, w), lin(q + "g2", H * dv, rank_g, 2.0)
            norm(q + "norm", dv, bias=False)
        if e["mlp"]:
            norm(p + "norm2", w)
            ff = e["mlp"]["ff"]
            lin(p + "mlp.gate", ff, w), lin(p + "mlp.up", ff, w), lin(p + "mlp.down", w, ff)
    return {k: bf16(v) for k, v in W.items()}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(1, cfg["vocab"], n).astype(np.int32)


class Case:
    """A configuration with its weights, and the oracle's logits of token lists (computed once each)."""

    make_weights, forward = staticmethod(weights), staticmethod(R.forward)

    def __init__(self, cfg, seed=0, edit=None, **kw):
        self.cfg, self.W = cfg, self.make_weights(cfg, seed, **kw)
        if edit:
            edit(self.W)
            self.W = {k: bf16(v) for k, v in self.W.items()}
        self._ref = {}

    def model(self, ctx, dtype="float32", max_rows=512):
        m = D.DecoderModel(ctx, registry.describe(self.cfg, lambda n: self.W[n].shape), dtype, max_rows)
        m.loadTensors(self.W.__getitem__)
        return m

    def ref(self, toks, cfg=None):
        key = (tuple(int(t) for t in toks), id(cfg))
        if key not in self._ref:
            self._ref[key] = self.forward(cfg or self.cfg, self.W, np.asarray(toks))
        return self._ref[key]


def error(got, want):
    """Per position: root mean square over the vocabulary of the difference (mean taken off), over that of the expected logits."""
    d = np.asarray(got, np.float64) - want
    d = d - d.mean(-1, keepdims=True)
    c = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((c * c).mean())


def run_steps(model, pool, plan):
    """plan: steps [[(name, tokens)], ...] -> {name: logits of all its tokens}; sequences are allocated at first sight and
    freed when the plan names them with None."""
    seqs, out = {}, {}
    for step in plan:
        go = [(n, t) for n, t in step if t is not None]
        for n, _ in go:
            if n not in seqs:
                seqs[n] = pool.seq_alloc()
        if go:
            rows = sum(len(t) for _, t in go)
            lg, _ = model.step(pool, [seqs[n] for n, _ in go], [t for _, t in go], np.arange(rows))
            at = 0
            for n, t in go:
                out.setdefault(n, []).append(lg[at:at + len(t)])
                at += len(t)
        for n, t in step:
            if t is None:
                pool.seq_free(seqs.pop(n))
    for s in seqs.values():
        pool.seq_free(s)
    return {n: np.concatenate(v) for n, v in out.items()}


def cut(toks, sizes):
    """Portions of the given sizes, the last size repeated to the end."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = sizes[min(i, len(sizes) - 1)]
        out.append(toks[at:at + n])
        at, i = at + n, i + 1
    return out


def mixed_plan(toks, seed, live=3):
    """Requests that start, pause, go on in portions or single tokens, and end: at most `live` at a time."""
    rng = np.random.default_rng(seed)
    at, active, todo, plan = {n: 0 for n in toks}, [], list(toks), []
    while todo or active:
        while todo and len(active) < live:
            active.append(todo.pop(0))
        step = []
        for n in list(active):
            if rng.random() < 0.2:
                continue  # left out of this step
            k = int(rng.choice([1, 1, 1, 2, 3, 16, 29, 64, 90]))
            step.append((n, toks[n][at[n]:at[n] + k]))
            at[n] += k
        for n in list(active):
            if at[n] >= len(toks[n]):
                active.remove(n)
                step.append((n, None))
        plan.append(step)
    return plan


def greedy(case, prompt, n):
    """The oracle's greedy continuation and the smallest margin between its best two logits."""
    out, margin = list(prompt), np.inf
    for _ in range(n):
        lg = case.forward(case.cfg, case.W, np.array(out))[-1]
        top = np.sort(lg)[-2:]
        margin = min(margin, top[1] - top[0])
        out.append(int(lg.argmax()))
        if out[-1] == 0:
            break
    return out[len(prompt):], margin
