"""Plain, slow restatement of the Lipelix design's mechanisms (numpy, float64): one function per mechanism, whole sequences
at once, no cache, no batching, a loop over heads and tokens.  Shares no code with the library.

Notation as in hybrid_ref: T tokens, D width, H query heads, G key heads, dk / dv head sizes; linear weights are [out, in].
"""
from __future__ import annotations

import numpy as np

from .hybrid_ref import F, linear, rms_norm, sigmoid, sub


# ---- rotation ---------------------------------------------------------------------------------------
def rotate(x, rot):
    """x [T, n, dk]; row t is at position t; element i of the first rot.dims turns with element i + rot.dims / 2."""
    n = rot["dims"]
    f = np.array([float(rot["base"]) ** (-2.0 * i / n) for i in range(n // 2)], F)
    y = np.array(x, F)
    for t in range(x.shape[0]):
        c, s = np.cos(t * f), np.sin(t * f)
        u, v = x[t, :, :n // 2], x[t, :, n // 2:n]
        y[t, :, :n // 2], y[t, :, n // 2:n] = u * c - v * s, v * c + u * s
    return y


# ---- attention --------------------------------------------------------------------------------------
def visible(T, mask=None):
    """[T, T] bool: which keys (columns) a query (row) sees: all earlier ones, or the last mask.size with the first mask.keep_first."""
    ok = np.zeros((T, T), bool)
    for i in range(T):
        for j in range(i + 1):
            ok[i, j] = mask is None or i - j < mask["size"] or j < mask["keep_first"]
    return ok


def sink_softmax(s, sink):
    """Weights over the last axis; the sink takes its share of the sum and goes nowhere."""
    top = np.maximum(s.max(-1, keepdims=True), sink)
    p = np.exp(s - top)
    return p / (p.sum(-1, keepdims=True) + np.exp(sink - top))


def attend(q, k, v, scale, ok, sinks):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv], sinks [H] -> [T, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    return np.stack([sink_softmax(np.where(ok, q[:, h] @ k[:, h * G // H].T * scale, -np.inf), sinks[h]) @ v[:, h * G // H] for h in range(H)], 1)


def mixed_values(v, first, share):
    """v, first [T, G * dv]; first is None in the layer that the values come from."""
    return v if first is None else (1 - share) * v + share * first


def heads(y, n):
    return y.reshape(y.shape[0], n, -1)


def projected_values(h, W, m, first):
    """Flat values [T, G * dv] as they are cached."""
    v = linear(h, W["v"])
    return mixed_values(v, first, W["vmix"]) if m.get("v_mix") else v


def normed_attention(h, W, m, eps, values):
    """Norm over all heads' rows at once, rotation, all earlier positions, a learned sink per head."""
    H, G = m["heads"], m["kv_heads"]
    q = rotate(heads(rms_norm(linear(h, W["q"]), W["q.norm"], eps), H), m["rot"])
    k = rotate(heads(rms_norm(linear(h, W["k"]), W["k.norm"], eps), G), m["rot"])
    o = attend(q, k, heads(values, G), m["scale"], visible(h.shape[0]), W["sink"])
    return linear(o.reshape(h.shape[0], -1), W["o"])


def windowed_attention(h, W, m, eps, values):
    """Rotation, then unit root mean square per head; a window and the first tokens; a sink of score 0."""
    H, G = m["heads"], m["kv_heads"]
    q = rms_norm(rotate(heads(linear(h, W["q"]), H), m["rot"]), 1.0, eps)
    k = rms_norm(rotate(heads(linear(h, W["k"]), G), m["rot"]), 1.0, eps)
    o = attend(q, k, heads(values, G), m["scale"], visible(h.shape[0], m["mask"]), np.zeros(H, F))
    return linear(o.reshape(h.shape[0], -1), W["o"])


# ---- generalised delta rule -------------------------------------------------------------------------------
def general_delta_scan(r, k, v, w, a):
    """S <- diag(w) S - (a u) (u^T S) + k v^T with the old S on the right and u = k / |k|; o = S^T r.  r, k, w, a [T, H, d], v [T, H, dv]."""
    T, H, d = r.shape
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        S = np.zeros((d, v.shape[2]), F)
        for t in range(T):
            u = k[t, h] / np.sqrt((k[t, h] ** 2).sum() + 1e-6)
            S = w[t, h][:, None] * S - np.outer(a[t, h] * u, u @ S) + np.outer(k[t, h], v[t, h])
            out[t, h] = r[t, h] @ S
    return out


def delta_decay(h, W):
    return np.exp(-np.exp(-0.5) * sigmoid(linear(np.tanh(linear(h, W["w1"])), W["w2"]) + W["w0"]))


def removal_rate(h, W):
    return sigmoid(linear(h, W["a"]) + W["a.b"])


def general_delta(h, W, m, eps):
    H = m["heads"]
    r, k, v = (heads(linear(h, W[n]), H) for n in "rkv")
    o = general_delta_scan(r, k, v, heads(delta_decay(h, W), H), heads(removal_rate(h, W), H))
    o = rms_norm(o, 1.0, eps).reshape(h.shape[0], -1) * W["norm"] * sigmoid(linear(h, W["g"]))
    return linear(o, W["o"])


# ---- the residual stream ----------------------------------------------------------------------------------
def shifted(h, share):
    """h + (h' - h) share, h' the row before (zeros in front of the first)."""
    before = np.concatenate([np.zeros((1, h.shape[1]), F), h[:-1]])
    return h + (before - h) * share


def gated(y, h, W, b):
    return y * sigmoid(linear(h, W) + b)


def dense_part(h, W):
    return linear(np.maximum(linear(h, W["up"]), 0) ** 2, W["down"])


# ---- the whole model ---------------------------------------------------------------------------------
def forward(cfg, W, tokens, layer_outputs=None):
    """Logits [T, vocab] of one sequence from its start; layer_outputs (a list) receives x after every layer."""
    W = {k: np.asarray(v, F) for k, v in W.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x, first = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"], None
    for i, layer in enumerate(cfg["layers"]):
        L, m = sub(W, f"l{i}."), layer["mixer"]
        M, h = sub(L, "mix."), rms_norm(x, L["norm1"], eps)
        s = shifted(h, L["shift"])
        if layer["type"] == "general_delta":
            y = general_delta(s, M, m, eps)
        else:
            values = projected_values(s, M, m, first)
            if m.get("v_mix") and first is None:
                first = values
            y = {"attention": normed_attention, "attention_2": windowed_attention}[layer["type"]](s, M, m, eps, values)
        x = x + mult * rms_norm(gated(y, h, L["rg1"], L["rg1.b"]), L["norm1b"], eps)
        if layer["mlp"] is not None:
            h = rms_norm(x, L["norm2"], eps)
            x = x + mult * rms_norm(gated(dense_part(h, sub(L, "mlp.")), h, L["rg2"], L["rg2.b"]), L["norm2b"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return linear(rms_norm(x, W["final.norm"], eps), W["head"])
