"""Plain, slow restatement of the Nefipel design's mechanisms (numpy, float64): one function per mechanism, whole sequences
at once, no cache, no batching, a loop over heads, maps and experts.  Shares no code with the library.

Notation as in hybrid_ref: T tokens, D width, H query heads, G key heads, dk / dv head sizes; linear weights are [out, in].
"""
from __future__ import annotations

import numpy as np

from .hybrid_ref import F, linear, rms_norm, sigmoid, sub


def relu(z):
    return np.maximum(z, 0)


# ---- rotation ---------------------------------------------------------------------------------------
def frequencies(rot):
    """(turns per position of every pair in radians, magnitude of cos and sin); with scaling, pairs that turn slowly over the
    original length are slowed down by the factor, fast ones are left alone, a linear ramp lies between."""
    n, base, s = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)], F)
    if not s:
        return f, 1.0

    def pair_of(turns):
        return n * np.log(s["original"] / (2 * np.pi * turns)) / (2 * np.log(base))
    lo, hi = max(np.floor(pair_of(s["fast"])), 0), min(np.ceil(pair_of(s["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0, 1)
    return ramp * f / s["factor"] + (1 - ramp) * f, 1 + 0.1 * np.log(s["factor"])


def rotate(x, rot, layout):
    """x [T, ..., dk]; row t is at position t.  'half': pairs (i, i + n / 2), 'interleaved': pairs (2 i, 2 i + 1)."""
    f, mag = frequencies(rot)
    n, y = rot["dims"], np.array(x, F)
    for t in range(x.shape[0]):
        c, s = np.cos(t * f) * mag, np.sin(t * f) * mag
        first = np.arange(n // 2) if layout == "half" else 2 * np.arange(n // 2)
        second = first + (n // 2 if layout == "half" else 1)
        u, v = x[t][..., first], x[t][..., second]
        y[t][..., first], y[t][..., second] = u * c - v * s, v * c + u * s
    return y


# ---- attention --------------------------------------------------------------------------------------
def causal_softmax_attention(q, k, v, scale):
    """One head: q, k [T, dk], v [T, dv]."""
    T = q.shape[0]
    s = np.where(np.tril(np.ones((T, T), bool)), q @ k.T * scale, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return (p / p.sum(-1, keepdims=True)) @ v


def projected(h, W, name):
    y = linear(h, W[name])
    return y + W[name + ".b"] if name + ".b" in W else y


def normed_heads(y, W, name, dim, eps, rot, layout):
    """[T, n * dim] -> [T, n, dim]: unit root mean square per head (or map of a head), its weight, rotation."""
    return rotate(rms_norm(y.reshape(y.shape[0], -1, dim), W[name + ".norm"], eps), rot, layout)


def gated_attention(h, W, m, eps):
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = normed_heads(projected(h, W, "q"), W, "q", dk, eps, m["rot"], "half")
    k = normed_heads(projected(h, W, "k"), W, "k", dk, eps, m["rot"], "half")
    v = projected(h, W, "v").reshape(T, G, dv)
    o = np.stack([causal_softmax_attention(q[:, i], k[:, i * G // H], v[:, i * G // H], m["scale"]) for i in range(H)], 1)
    return linear(o.reshape(T, -1) * sigmoid(linear(h, W["g"])), W["o"])


def difference_factor(W, diff):
    return np.exp((W["lq1"] * W["lk1"]).sum()) - np.exp((W["lq2"] * W["lk2"]).sum()) + diff


def differential_attention(h, W, m, eps):
    """Two attention maps per head over the same values; the second one's output is taken off the first one's."""
    T, H, G, dk, dv, diff = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["diff"]
    q = normed_heads(projected(h, W, "q"), W, "q", dk, eps, m["rot"], "interleaved").reshape(T, H, 2, dk)
    k = normed_heads(projected(h, W, "k"), W, "k", dk, eps, m["rot"], "interleaved").reshape(T, G, 2, dk)
    v = projected(h, W, "v").reshape(T, G, dv)
    factor, o = difference_factor(W, diff), np.zeros((T, H, dv), F)
    for i in range(H):
        g = i * G // H
        a1, a2 = (causal_softmax_attention(q[:, i, j], k[:, g, j], v[:, g], m["scale"]) for j in range(2))
        o[:, i] = rms_norm(a1 - factor * a2, 1.0, eps) * (1 - diff)
    return linear(o.reshape(T, -1), W["o"])


# ---- feed-forward -----------------------------------------------------------------------------------
def dense_part(h, W):
    return linear(relu(linear(h, W["gate"])) * linear(h, W["up"]), W["down"])


def expert(h, up, down):
    return linear(relu(linear(h, up)) ** 2, down)


def open_groups(choice, r):
    """Which outputs may be chosen: those of the groups whose best choice score is among the largest."""
    g = r.get("groups") or {"count": 1, "keep": 1}
    size = choice.size // g["count"]
    best = np.argsort(-choice.reshape(g["count"], size).max(1), kind="stable")[:g["keep"]]
    return np.isin(np.arange(choice.size) // size, best)


def route(z, correction, r):
    """One token: router logits -> [(expert, weight)]; the correction takes part in the choice only."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    choice = s + correction
    chosen = np.argsort(-np.where(open_groups(choice, r), choice, -np.inf), kind="stable")[:r["top"]]
    return [(int(e), s[e] / (s[chosen].sum() + 1e-20)) for e in chosen]


def route_margin(z, correction, r):
    """How far one choice score is from changing what is chosen."""
    s = np.exp(z - z.max())
    choice = s / s.sum() + correction
    ok, g = open_groups(choice, r), r.get("groups") or {"count": 1, "keep": 1}
    inside, best = -np.sort(-choice[ok]), -np.sort(-choice.reshape(g["count"], -1).max(1))
    gaps = [inside[r["top"] - 1] - inside[r["top"]]] if inside.size > r["top"] else []
    gaps += [best[g["keep"] - 1] - best[g["keep"]]] if g["keep"] < g["count"] else []
    return min(gaps, default=np.inf)


def mixture(h, W, mlp):
    r, out = mlp["router"], np.zeros_like(h)
    z = linear(h, W["router"])
    for t in range(h.shape[0]):
        for e, w in route(z[t], W["correction"], r):
            out[t] += w * (expert(h[t], W[f"e{e}.up"], W[f"e{e}.down"]) if e < r["experts"] else h[t])
    if mlp.get("shared"):
        out = out + sigmoid(linear(h, W["shared.sg"])) * expert(h, W["shared.up"], W["shared.down"])
    return out


# ---- the whole model ---------------------------------------------------------------------------------
def forward(cfg, W, tokens, layer_outputs=None):
    """Logits [T, vocab] of one sequence from its start; layer_outputs (a list) receives x after every layer."""
    W = {k: np.asarray(v, F) for k, v in W.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        L = sub(W, f"l{i}.")
        mixer = {"attention": gated_attention, "attention_2": differential_attention}[layer["type"]]
        x = rms_norm(alpha * x + mixer(x, sub(L, "mix."), layer["mixer"], eps), L["norm1"], eps)
        mlp = layer["mlp"]
        if mlp is not None:
            M = sub(L, "mlp.")
            y = dense_part(x, M) if mlp["kind"] == "dense" else mixture(x, M, mlp)
            x = rms_norm(alpha * x + y, L["norm2"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return linear(rms_norm(x, W["final.norm"], eps), W["embed"])
