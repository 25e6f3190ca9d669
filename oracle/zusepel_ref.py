"""Plain, slow restatement of the Zusepel design's mechanisms (numpy, float64): one function per mechanism, whole sequences
at once, no cache, no batching, keys and values written out per head.  Shares no code with the library.

Notation as in hybrid_ref: T tokens, D width, H heads, dk / dv head sizes; linear weights are [out, in].
"""
from __future__ import annotations

import numpy as np

from .hybrid_ref import F, gla_scan, linear, rms_norm, sigmoid, silu, softplus, sub


# ---- rotation ---------------------------------------------------------------------------------------
def yarn_frequencies(dims, base, scaling=None):
    """(frequencies [dims / 2], magnitude of cos and sin).  Slow dimensions (few turns over the original length) are slowed
    down by the factor, fast ones stay, a linear ramp lies between."""
    i = np.arange(dims // 2, dtype=F)
    f = float(base) ** (-2.0 * i / dims)
    if scaling is None:
        return f, 1.0

    def dim_of(turns):
        return dims * np.log(scaling["original"] / (2 * np.pi * turns)) / (2 * np.log(float(base)))
    lo = max(np.floor(dim_of(scaling["fast"])), 0)
    hi = min(np.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0, 1)
    return f / scaling["factor"] * ramp + f * (1 - ramp), 0.1 * np.log(scaling["factor"]) + 1.0


def rotate_half(x, positions, rot):
    """x [T, ..., n]: dimension i of the first rot.dims is turned with dimension i + rot.dims / 2."""
    f, mag = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    a = np.asarray(positions, F)[:, None] * f
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (f.size,)
    c, s = (np.cos(a) * mag).reshape(shape), (np.sin(a) * mag).reshape(shape)
    n = f.size
    u, v = x[..., :n], x[..., n:2 * n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


# ---- latent attention inside a sliding window ----------------------------------------------------------
def window_visible(T, size):
    """[T, T] bool: query i sees the size keys that end with its own."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < size)


def softmax_attention(q, k, v, scale, visible):
    """q, k [T, H, dk], v [T, H, dv] -> [T, H, dv]."""
    out = np.zeros((q.shape[0],) + v.shape[1:], F)
    for h in range(q.shape[1]):
        s = np.where(visible, q[:, h] @ k[:, h].T * scale, -np.inf)
        p = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = (p / p.sum(-1, keepdims=True)) @ v[:, h]
    return out


def latent_keys(h, W, m, eps):
    """What a layer's cache holds: (latent [T, kv_rank], rotated key part [T, rot_dim])."""
    z = linear(h, W["dkv"])
    r = m["kv_rank"]
    return rms_norm(z[:, :r], np.asarray(W["dkv.norm"], F), eps), rotate_half(z[:, r:], np.arange(h.shape[0]), m["rot"])


def latent_queries(h, W, m, eps):
    T = h.shape[0]
    q = linear(rms_norm(linear(h, W["dq"]), np.asarray(W["dq.norm"], F), eps), W["uq"]).reshape(T, m["heads"], m["dim"] + m["rot_dim"])
    return np.concatenate([q[..., :m["dim"]], rotate_half(q[..., m["dim"]:], np.arange(T), m["rot"])], -1)


def latent_attention(h, W, m, eps, cached):
    T, H = h.shape[0], m["heads"]
    c, kr = cached
    k = np.concatenate([linear(c, W["uk"]).reshape(T, H, m["dim"]), np.broadcast_to(kr[:, None], (T, H, kr.shape[1]))], -1)
    v = linear(c, W["uv"]).reshape(T, H, m["vdim"])
    o = softmax_attention(latent_queries(h, W, m, eps), k, v, m["scale"], window_visible(T, m["mask"]["size"]))
    return linear(o.reshape(T, -1), W["o"])


# ---- recurrences ----------------------------------------------------------------------------------------
def token_shift(h):
    return np.concatenate([np.zeros((1, h.shape[1]), F), h[:-1]])


def wkv_scan(r, k, v, w, u):
    """o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T per head; r, k, w [T, H, d], v [T, H, dv], u [H, d]."""
    T, H, d = r.shape
    S = np.zeros((H, d, v.shape[2]), F)
    out = np.zeros((T, H, v.shape[2]), F)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return out


def wkv_decay(mixed, W, heads, dim):
    y = linear(np.tanh(linear(mixed, W["w1"])), W["w2"]) + np.asarray(W["w0"], F)
    return np.exp(-np.exp(y)).reshape(mixed.shape[0], heads, dim)


def wkv_mixer(h, W, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    prev = token_shift(h)
    mix = {s: h + (prev - h) * np.asarray(W["mu." + s], F) for s in "rkvgw"}
    r, k, v = (linear(mix[s], W[s]).reshape(T, H, d) for s in "rkv")
    o = wkv_scan(r, k, v, wkv_decay(mix["w"], W, H, d), np.asarray(W["u"], F))
    o = rms_norm(o, 1.0, eps).reshape(T, H * d) * np.asarray(W["norm"], F) * silu(linear(mix["g"], W["g"]))
    return linear(o, W["o"])


def hgrn2_forget(h, W):
    low = np.asarray(W["lower"], F)
    return low + (1 - low) * sigmoid(linear(h, W["f"]) + np.asarray(W["f.b"], F))


def hgrn2_mixer(h, W, m, eps):
    """S <- diag(f) S + (1 - f) v^T, o = S^T q."""
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    f = hgrn2_forget(h, W).reshape(T, H, dk)
    q, v = silu(linear(h, W["q"])).reshape(T, H, dk), linear(h, W["v"]).reshape(T, H, dv)
    o = rms_norm(gla_scan(q, 1 - f, v, f), np.asarray(W["norm"], F), eps)
    return linear(o.reshape(T, -1), W["o"])


# ---- feed-forward -----------------------------------------------------------------------------------------
def xielu(z, p, q):
    neg = np.minimum(z, 0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + z / 2


# ---- the whole model ---------------------------------------------------------------------------------------
def depth_average(weights, outputs):
    return sum(w * x for w, x in zip(weights, outputs, strict=True))


def forward(cfg, W, tokens, layer_outputs=None):
    """Logits [T, vocab] of one sequence from its start; layer_outputs (a list) receives x after every layer."""
    W = {k: np.asarray(v, F) for k, v in W.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][np.asarray(tokens)]
    results, caches = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        L, m = sub(W, f"l{i}."), layer["mixer"]
        M, h = sub(L, "mix."), rms_norm(x, L["norm1"], eps)
        if layer["type"] == "latent_attention":
            source = m.get("kv_from")
            if source is None:
                caches[i] = latent_keys(h, M, m, eps)
            y = latent_attention(h, M, m, eps, caches[i if source is None else source])
        else:
            y = {"wkv": wkv_mixer, "hgrn2": hgrn2_mixer}[layer["type"]](h, M, m, eps)
        x = x + mult * (L["ls1"] * y)
        if layer["mlp"] is not None:
            z = linear(rms_norm(x, L["norm2"], eps), L["mlp.up"])
            x = x + mult * (L["ls2"] * linear(xielu(z, *L["mlp.act"]), L["mlp.down"]))
        results.append(x)
        x = depth_average(L["dwa"], results)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return linear(rms_norm(x, W["final.norm"], eps), W["head"])
