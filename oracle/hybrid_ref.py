"""Plain, slow restatement of the layered-decoder mechanisms (numpy, float64): one function per mechanism, whole
sequences at once, no cache, no batching.  The library's kernels and state manager are compared with it; it shares no
code with them.

Notation: T tokens, D width, H query / value heads, G key heads, dk / dv head sizes.  Linear weights are [out, in].
"""
from __future__ import annotations

import numpy as np

F = np.float64


# ---- elementwise ------------------------------------------------------------------------------------
def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, F)))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, np.asarray(z, F))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdims=True)
    return c / np.sqrt((c * c).mean(-1, keepdims=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def linear(x, w):
    return x @ np.asarray(w, F).T


# ---- embedding and output -----------------------------------------------------------------------------
def embed(tokens, table, pos_table, scale, w, b, eps):
    tokens = np.asarray(tokens)
    x = np.asarray(table, F)[tokens] * scale + np.asarray(pos_table, F)[np.arange(tokens.size)]
    return layer_norm(x, np.asarray(w, F), np.asarray(b, F), eps)


def tied_logits(x, table, w, b, eps, logit_scale):
    return linear(layer_norm(x, np.asarray(w, F), np.asarray(b, F), eps), table) * logit_scale


# ---- attention over the positions of the query's own chunk ---------------------------------------------
def chunk_visible(T, chunk):
    """[T, T] bool: query i sees key j.  chunk <= 0: plain causal."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    ok = j <= i
    return ok if chunk <= 0 else ok & (i // chunk == j // chunk)


def attention(q, k, v, scale, chunk):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]; query head h reads key head h // (H / G)."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    ok = chunk_visible(T, chunk)
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        s = q[:, h] @ k[:, h // rep].T * scale
        s = np.where(ok, s, -np.inf)
        p = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = (p / p.sum(-1, keepdims=True)) @ v[:, h // rep]
    return out


def gated_chunk_attention(h, W, m):
    """W: q, k, v, g, o by name; m: heads, kv_heads, dim, vdim, scale, mask.size."""
    T = h.shape[0]
    q = linear(h, W["q"]).reshape(T, m["heads"], m["dim"])
    k = linear(h, W["k"]).reshape(T, m["kv_heads"], m["dim"])
    v = linear(h, W["v"]).reshape(T, m["kv_heads"], m["vdim"])
    o = attention(q, k, v, m["scale"], m["mask"]["size"]) * sigmoid(linear(h, W["g"]))[:, :, None]
    return linear(o.reshape(T, -1), W["o"])


# ---- gated linear attention ------------------------------------------------------------------------------
def gla_scan(q, k, v, alpha):
    """S <- diag(alpha) S + k v^T, o = S^T q per head; q, k, alpha [T, H, dk], v [T, H, dv]."""
    T, H, dk = q.shape
    S = np.zeros((H, dk, v.shape[2]), F)
    out = np.zeros((T, H, v.shape[2]), F)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S, q[t])
    return out


def gla_decay(h, W, heads, dim, tau):
    z = linear(linear(h, W["a1"]), W["a2"]) + np.asarray(W["a2.b"], F)
    return (sigmoid(z) ** (1.0 / tau)).reshape(h.shape[0], heads, dim)


def gated_linear_attention(h, W, m, eps):
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(h, W["q"]).reshape(T, H, dk) * dk ** -0.5
    k = linear(h, W["k"]).reshape(T, H, dk)
    v = linear(h, W["v"]).reshape(T, H, dv)
    o = gla_scan(q, k, v, gla_decay(h, W, H, dk, m["tau"]))
    o = rms_norm(o, np.asarray(W["norm"], F), eps).reshape(T, H * dv) * silu(linear(h, W["g"]))
    return linear(o, W["o"])


# ---- gated delta rule with a decay per key channel -------------------------------------------------------
def short_conv(x, w):
    """Causal convolution per channel, last column of w = the current token; x [T, C], w [C, taps]."""
    w = np.asarray(w, F)
    taps = w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, x.shape[1]), F), x])
    return sum(pad[i:i + x.shape[0]] * w[:, i] for i in range(taps))


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def delta_decay(h, W, heads, dim):
    z = linear(linear(h, W["a1"]), W["a2"]) + np.asarray(W["dt_bias"], F)
    rate = np.exp(np.asarray(W["A_log"], F))[:, None]
    return np.exp(-rate * softplus(z.reshape(h.shape[0], heads, dim)))


def delta_scan(q, k, v, g, beta):
    """S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q; q, k, g [T, H, dk], v [T, H, dv], beta [T, H]."""
    T, H, dk = q.shape
    S = np.zeros((H, dk, v.shape[2]), F)
    out = np.zeros((T, H, v.shape[2]), F)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S, q[t])
    return out


def channel_delta(h, W, m, eps):
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_conv(linear(h, W["q"]), W["q.conv"])).reshape(T, G, dk)
    k = silu(short_conv(linear(h, W["k"]), W["k.conv"])).reshape(T, G, dk)
    v = silu(short_conv(linear(h, W["v"]), W["v.conv"])).reshape(T, H, dv)
    q, k = np.repeat(unit(q) * dk ** -0.5, H // G, 1), np.repeat(unit(k), H // G, 1)
    o = delta_scan(q, k, v, delta_decay(h, W, H, dk), sigmoid(linear(h, W["b"])))
    gate = sigmoid(linear(linear(h, W["g1"]), W["g2"])).reshape(T, H, dv)
    o = rms_norm(o, np.asarray(W["norm"], F), eps) * gate
    return linear(o.reshape(T, -1), W["o"])


# ---- the whole model ---------------------------------------------------------------------------------------
def sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def mixer(kind, h, W, m, eps):
    if kind == "channel_delta":
        return channel_delta(h, W, m, eps)
    if kind == "parallel":
        return (m["left_scale"] * gated_chunk_attention(h, sub(W, "left."), m["left"])
                + m["right_scale"] * gated_linear_attention(h, sub(W, "right."), m["right"], eps))
    raise ValueError(f"unknown mixer {kind}")


def forward(cfg, W, tokens, layer_outputs=None):
    """Logits [T, vocab] of one sequence from its start; layer_outputs (a list) receives x after every layer."""
    W = {k: np.asarray(v, F) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, W["embed"], W["pos"], cfg["embedding"]["scale"], W["embed.norm"], W["embed.norm.b"], eps)
    for i, layer in enumerate(cfg["layers"]):
        L = sub(W, f"l{i}.")
        x = x + mixer(layer["type"], layer_norm(x, L["norm1"], L["norm1.b"], eps), sub(L, "mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            h = layer_norm(x, L["norm2"], L["norm2.b"], eps)
            x = x + linear(gelu_tanh(linear(h, L["mlp.gate"])) * linear(h, L["mlp.up"]), L["mlp.down"])
        if layer_outputs is not None:
            layer_outputs.append(x)
    return tied_logits(x, W["embed"], W["final.norm"], W["final.norm.b"], eps, cfg["logit_scale"])
