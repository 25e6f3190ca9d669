"""Small models of the Zusepel design with random weights: configurations, weights, and what the tests need to build the
library's model from them."""
from __future__ import annotations

import numpy as np

import decoder_cases as dc
from oracle import zusepel_ref as Z

YARN = {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}


def latent(heads=3, dim=20, rot_dim=12, vdim=28, q_rank=36, kv_rank=44, size=40, scale=None, base=300.0, yarn=YARN, kv_from=None, ff=52):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "mask": {"size": size},
         "rot": {"base": base, "dims": rot_dim}, "scale": scale or 1.3 * (dim + rot_dim) ** -0.5}
    if yarn:
        m["rot"]["scaling"] = yarn
    if kv_from is not None:
        m["kv_from"] = kv_from
    return _layer("latent_attention", m, ff)


def wkv(heads=3, dim=24, ff=44):
    return _layer("wkv", {"heads": heads, "dim": dim}, ff)


def hgrn2(heads=2, dim=20, vdim=36, ff=60):
    return _layer("hgrn2", {"heads": heads, "dim": dim, "vdim": vdim}, ff)


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=72, vocab=101, eps=3e-6, mult=0.8):
    return {"architecture": "Zusepel", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult}


def weights(cfg, seed=0, rank=10):
    rng = np.random.default_rng(seed)
    W, w = {}, cfg["width"]

    def lin(name, out, inp, gain=1.0):
        W[name] = rng.standard_normal((out, inp)) * gain / np.sqrt(inp)

    def vec(name, n, at=1.0, by=0.2):
        W[name] = at + by * rng.standard_normal(n)
    W["embed"] = rng.standard_normal((cfg["vocab"], w))
    lin("head", cfg["vocab"], w), vec("final.norm", w)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        vec(p + "norm1", w), vec(p + "ls1", w, 0.9)
        W[p + "dwa"] = np.append(0.15 * rng.standard_normal(i + 1), 0.9 + 0.2 * rng.random())
        q, H, d = p + "mix.", m["heads"], m["dim"]
        if e["type"] == "latent_attention":
            lin(q + "dq", m["q_rank"], w), vec(q + "dq.norm", m["q_rank"]), lin(q + "uq", H * (d + m["rot_dim"]), m["q_rank"], 1.5)
            if "kv_from" not in m:
                lin(q + "dkv", m["kv_rank"] + m["rot_dim"], w), vec(q + "dkv.norm", m["kv_rank"])
            lin(q + "uk", H * d, m["kv_rank"], 1.5), lin(q + "uv", H * m["vdim"], m["kv_rank"]), lin(q + "o", w, H * m["vdim"])
        elif e["type"] == "wkv":
            for s in "rkvgw":
                W[q + "mu." + s] = rng.random(w)
            for s in "rkvg":
                lin(q + s, H * d, w)
            lin(q + "w1", rank, w), lin(q + "w2", H * d, rank), vec(q + "w0", H * d, -2.5, 1.5)
            W[q + "u"] = 0.5 * rng.standard_normal((H, d))
            vec(q + "norm", H * d), lin(q + "o", w, H * d)
        else:
            for s in "qf":
                lin(q + s, H * d, w)
            vec(q + "f.b", H * d, 2.0, 1.5)
            W[q + "lower"] = 0.9 * rng.random(H * d)
            lin(q + "v", H * m["vdim"], w), vec(q + "norm", m["vdim"]), lin(q + "o", w, H * m["vdim"])
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            vec(p + "norm2", w), vec(p + "ls2", w, 0.9)
            lin(p + "mlp.up", ff, w), lin(p + "mlp.down", w, ff)
            W[p + "mlp.act"] = rng.standard_normal(2) * 0.6 - 0.5
    return {k: dc.bf16(v) for k, v in W.items()}


class Case(dc.Case):
    make_weights, forward = staticmethod(weights), staticmethod(Z.forward)
