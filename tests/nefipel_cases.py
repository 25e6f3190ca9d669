"""Small models of the Nefipel design with random weights: configurations, weights, and what the tests need to build the
library's model from them."""
from __future__ import annotations

import numpy as np

import decoder_cases as dc
from oracle import nefipel_ref as N

YARN = {"factor": 3.0, "original": 60, "fast": 8.0, "slow": 1.0}


def dense(ff=44):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, identity=1, top=3, count=2, keep=1, ff=28, shared=36):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": count, "keep": keep}}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def att(heads=6, kv_heads=2, dim=20, vdim=12, rot_dims=None, base=300.0, scale=None, mlp="dense"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims},
         "scale": scale or 1.2 * dim ** -0.5}
    return {"type": "attention", "mixer": m, "mlp": dense() if mlp == "dense" else mlp}


def diff(heads=4, kv_heads=2, dim=14, vdim=26, rot_dims=None, base=500.0, yarn=YARN, scale=None, at=0.4, mlp="moe"):
    e = att(heads, kv_heads, dim, vdim, rot_dims, base, scale, moe() if mlp == "moe" else mlp)
    e["mixer"]["diff"] = at
    if yarn:
        e["mixer"]["rot"]["scaling"] = yarn
    return {**e, "type": "attention_2"}


def config(layers, width=72, vocab=101, eps=3e-6, alpha=2.2, scale=7.0):
    return {"architecture": "Nefipel", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"scale": scale}}


def weights(cfg, seed=0, settled=False, sharp=1.0):
    """settled: corrections so far apart that rounding cannot change a choice (a choice is a jump, rounded models differ there);
    sharp: factor on the query norms."""
    rng = np.random.default_rng(seed)
    W, w = {}, cfg["width"]

    def lin(name, out, inp, gain=1.0):
        W[name] = rng.standard_normal((out, inp)) * gain / np.sqrt(inp)

    def vec(name, n, at=1.0, by=0.2):
        W[name] = at + by * rng.standard_normal(n)
    W["embed"] = rng.standard_normal((cfg["vocab"], w)) / np.sqrt(w)
    vec("final.norm", w)
    for i, e in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", e["mixer"], e["mlp"]
        q, H, G, d, v = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        maps = 2 if e["type"] == "attention_2" else 1
        vec(p + "norm1", w)
        lin(q + "q", H * maps * d, w), lin(q + "k", G * maps * d, w), lin(q + "v", G * v, w), lin(q + "o", w, H * v, 2.0)
        vec(q + "q.norm", d, sharp, 0.3 * sharp), vec(q + "k.norm", d, 1.0, 0.3)
        if maps == 1:
            for n, k in (("q.b", H * d), ("k.b", G * d), ("v.b", G * v)):
                vec(q + n, k, 0.0, 0.5)
            lin(q + "g", H * v, w, 1.5)
        else:
            for n in ("lq1", "lk1", "lq2", "lk2"):
                vec(q + n, d, 0.0, 0.3)
        if mlp is None:
            continue
        vec(p + "norm2", w)
        if mlp["kind"] == "dense":
            lin(p + "mlp.gate", mlp["ff"], w), lin(p + "mlp.up", mlp["ff"], w), lin(p + "mlp.down", w, mlp["ff"], 2.0)
            continue
        r = mlp["router"]
        n = r["experts"] + r["identity"]
        lin(p + "mlp.router", n, w, 1.5)
        W[p + "mlp.correction"] = rng.permutation(n) * 2.0 - n if settled else 0.1 * rng.standard_normal(n) - 0.05
        for k in range(r["experts"]):
            lin(p + f"mlp.e{k}.up", mlp["expert"]["ff"], w), lin(p + f"mlp.e{k}.down", w, mlp["expert"]["ff"], 2.0)
        if mlp.get("shared"):
            f = mlp["shared"]["ff"]
            lin(p + "mlp.shared.up", f, w), lin(p + "mlp.shared.down", w, f), lin(p + "mlp.shared.sg", 1, w, 1.5)
    return {k: dc.bf16(v) for k, v in W.items()}


class Case(dc.Case):
    make_weights, forward = staticmethod(weights), staticmethod(N.forward)
