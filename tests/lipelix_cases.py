"""Small models of the Lipelix design with random weights: configurations, weights, and what the tests need to build the
library's model from them."""
from __future__ import annotations

import numpy as np

import decoder_cases as dc
from oracle import lipelix_ref as L


def dense(ff=44):
    return {"kind": "dense", "ff": ff}


def att(heads=6, kv_heads=2, dim=20, vdim=12, rot_dims=None, base=300.0, scale=None, v_mix=True, mlp="dense"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims},
         "scale": scale or 1.2 * dim ** -0.5, "v_mix": v_mix}
    return {"type": "attention", "mixer": m, "mlp": dense() if mlp == "dense" else mlp}


def win(heads=4, kv_heads=2, dim=14, vdim=12, rot_dims=None, base=500.0, scale=None, v_mix=True, size=21, keep=5, mlp="dense"):
    e = att(heads, kv_heads, dim, vdim, rot_dims, base, scale or 1.5 * dim ** -0.5, v_mix, mlp)
    e["mixer"]["mask"] = {"size": size, "keep_first": keep}
    return {**e, "type": "attention_2"}


def gen(heads=3, dim=20, mlp=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def config(layers, width=72, vocab=101, eps=3e-6, mult=0.6, scale=2.0):
    return {"architecture": "Lipelix", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": scale}}


def weights(cfg, seed=0, rank=6):
    rng = np.random.default_rng(seed)
    W, w, source = {}, cfg["width"], False

    def lin(name, out, inp, gain=1.0):
        W[name] = rng.standard_normal((out, inp)) * gain / np.sqrt(inp)

    def vec(name, n, at=1.0, by=0.2):
        W[name] = at + by * rng.standard_normal(n)
    W["embed"] = rng.standard_normal((cfg["vocab"], w))
    vec("final.norm", w), lin("head", cfg["vocab"], w)
    for i, e in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", e["mixer"], e["mlp"]
        q = p + "mix."
        vec(p + "norm1", w), vec(p + "norm1b", w), vec(p + "shift", w, 0.4, 0.4), lin(p + "rg1", w, w), vec(p + "rg1.b", w, 0.3, 0.5)
        if e["type"] == "general_delta":
            n = m["heads"] * m["dim"]
            for k in "rkvga":
                lin(q + k, n, w)
            W[q + "r"] = 0.7 * (W[q + "r"] + W[q + "k"])  # a first token's output is (r . k) v brought to unit size: r . k stays away from 0
            vec(q + "a.b", n, 0.0, 0.7), vec(q + "w0", n, -1.0, 1.5), vec(q + "norm", n)
            lin(q + "w1", rank, w), lin(q + "w2", n, rank, 2.0), lin(q + "o", w, n)
        else:
            H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            lin(q + "q", H * d, w), lin(q + "k", G * d, w), lin(q + "v", G * v, w), lin(q + "o", w, H * v)
            if e["type"] == "attention":
                vec(q + "q.norm", H * d, 1.0, 0.3), vec(q + "k.norm", G * d, 1.0, 0.3), vec(q + "sink", H, 0.5, 1.0)
            if m["v_mix"]:
                W[q + "vmix"] = np.array(0.3 + 0.3 * rng.random())
                if not source:
                    W[q + "vmix"], source = np.array(7.0), True  # nobody reads it
        if mlp is None:
            continue
        vec(p + "norm2", w), vec(p + "norm2b", w), lin(p + "rg2", w, w), vec(p + "rg2.b", w, 0.3, 0.5)
        lin(p + "mlp.up", mlp["ff"], w), lin(p + "mlp.down", w, mlp["ff"])
    return {k: dc.bf16(v).reshape(np.shape(v)) for k, v in W.items()}


class Case(dc.Case):
    make_weights, forward = staticmethod(weights), staticmethod(L.forward)
