"""Prefill and decode throughput of the layered designs (Lipelix, Nefipel, Zusepel, Somopel; random weights) beside the fixed-block GPT model at
equal width, depth, feed-forward parameters and vocabulary: ``bench.py --workload decoder``."""
from __future__ import annotations

import time

import numpy as np

from . import decoder as D
from . import registry
from .model import GPTModel
from .runtime import Event

VOCAB, LAYERS, MAX_POS = 32000, 6, 2304


def somopel_config(width):
    h = width // 128
    par = {"type": "parallel", "mlp": {"kind": "dense", "ff": width * 11 // 4},
           "mixer": {"left": {"heads": h, "kv_heads": max(h // 4, 1), "dim": 128, "vdim": 128, "mask": {"size": 512}, "scale": 128 ** -0.5},
                     "right": {"heads": h, "dim": 64, "vdim": 128, "tau": 16.0}, "left_scale": 0.7, "right_scale": 0.9}}
    delta = {"type": "channel_delta", "mlp": {"kind": "dense", "ff": width * 11 // 4},
             "mixer": {"heads": h, "kv_heads": h, "dim": 128, "vdim": 128, "conv": 4}}
    return {"architecture": "Somopel", "width": width, "vocab": VOCAB, "max_positions": MAX_POS, "norm": {"eps": 1e-5},
            "layers": [delta, par, par] * (LAYERS // 3), "embedding": {"scale": 1.0}, "logit_scale": 0.5}


def random_somopel(ctx, width, max_rows, rank=64):
    cfg = somopel_config(width)
    rng = np.random.default_rng(0)
    shapes = {}

    def lin(n, o, i):
        shapes[n] = (o, i)

    def vec(n, k):
        shapes[n] = (k,)
    for n in ("embed.norm", "embed.norm.b", "final.norm", "final.norm.b"):
        vec(n, width)
    lin("embed", VOCAB, width), lin("pos", MAX_POS, width)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        for n in ("norm1", "norm1.b", "norm2", "norm2.b"):
            vec(p + n, width)
        ff = e["mlp"]["ff"]
        lin(p + "mlp.gate", ff, width), lin(p + "mlp.up", ff, width), lin(p + "mlp.down", width, ff)
        if e["type"] == "parallel":
            a, b = m["left"], m["right"]
            for n, k in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"]), ("g", a["heads"])):
                lin(p + "mix.left." + n, k, width)
            lin(p + "mix.left.o", width, a["heads"] * a["vdim"])
            q, hk, hv = p + "mix.right.", b["heads"] * b["dim"], b["heads"] * b["vdim"]
            lin(q + "q", hk, width), lin(q + "k", hk, width), lin(q + "v", hv, width), lin(q + "g", hv, width), lin(q + "o", width, hv)
            lin(q + "a1", rank, width), lin(q + "a2", hk, rank), vec(q + "a2.b", hk), vec(q + "norm", b["vdim"])
        else:
            q, H, G, dk, dv, t = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, k in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                lin(q + n, k, width), lin(q + n + ".conv", k, t)
            lin(q + "b", H, width), vec(q + "A_log", H), vec(q + "dt_bias", H * dk), lin(q + "o", width, H * dv)
            lin(q + "a1", rank, width), lin(q + "a2", H * dk, rank), lin(q + "g1", rank, width), lin(q + "g2", H * dv, rank), vec(q + "norm", dv)
    return _random_model(ctx, cfg, shapes, max_rows)


def _random_model(ctx, cfg, shapes, max_rows, seed=0):
    rng = np.random.default_rng(seed)
    noise = rng.standard_normal(1 << 22, dtype=np.float32)

    def get(n):  # slices of one noise block: making fresh numbers for every weight takes longer than the benchmark
        s = shapes[n]
        k = int(np.prod(s))
        x = np.resize(noise[int(rng.integers(0, 1 << 20)):], k).reshape(s)
        if n.endswith(".lower"):
            return 0.5 + 0.1 * np.tanh(x)
        if n.endswith(".w0"):
            return x - 4
        if n.endswith(".correction"):
            return 0.005 * x
        if n.endswith((".shift", ".vmix")):
            return 0.3 + 0.1 * np.tanh(x)
        if n.endswith((".a.b", ".rg1.b", ".rg2.b", ".q.b", ".k.b", ".v.b", ".lq1", ".lk1", ".lq2", ".lk2")):
            return 0.1 * x
        return x / np.sqrt(s[1]) if len(s) == 2 else 1 + 0.1 * x
    model = D.DecoderModel(ctx, registry.describe(cfg, shapes.__getitem__), "bfloat16", max_rows)
    model.loadTensors(get)
    return model


def zusepel_config(width):
    """Latent attention with 128 + 64 / 128 heads on a latent of 512 (window 512), WKV heads of 64, HGRN2 heads of 128."""
    h, mlp = width // 128, {"kind": "dense", "ff": width * 33 // 8}  # as many parameters as a gated part of 11 / 4
    rot = {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    latent = {"heads": h, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": width * 3 // 8, "kv_rank": 512, "mask": {"size": 512}, "rot": rot,
              "scale": 192 ** -0.5}
    block = [("latent_attention", latent), ("wkv", {"heads": 2 * h, "dim": 64}), ("hgrn2", {"heads": h, "dim": 128, "vdim": 128})]
    layers = [{"type": t, "mixer": m, "mlp": mlp} for t, m in block * (LAYERS // 3)]
    layers[3] = {**layers[3], "mixer": {**latent, "kv_from": 0}}
    return {"architecture": "Zusepel", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-6}, "residual_mult": 0.9, "layers": layers}


def random_zusepel(ctx, width, max_rows, rank=64):
    cfg = zusepel_config(width)
    shapes = {"embed": (VOCAB, width), "head": (VOCAB, width), "final.norm": (width,)}
    for i, e in enumerate(cfg["layers"]):
        p, m, ff = f"l{i}.", e["mixer"], e["mlp"]["ff"]
        new = {n: (width,) for n in ("norm1", "norm2", "ls1", "ls2")}
        new.update({"dwa": (i + 2,), "mlp.up": (ff, width), "mlp.down": (width, ff), "mlp.act": (2,)})
        H, d = m["heads"], m["dim"]
        if e["type"] == "latent_attention":
            r, v = m["rot_dim"], m["vdim"]
            new.update({"mix.dq": (m["q_rank"], width), "mix.dq.norm": (m["q_rank"],), "mix.uq": (H * (d + r), m["q_rank"]), "mix.uk": (H * d, m["kv_rank"]),
                        "mix.uv": (H * v, m["kv_rank"]), "mix.o": (width, H * v)})
            if "kv_from" not in m:
                new.update({"mix.dkv": (m["kv_rank"] + r, width), "mix.dkv.norm": (m["kv_rank"],)})
        elif e["type"] == "wkv":
            new.update({f"mix.mu.{s}": (width,) for s in "rkvgw"})
            new.update({f"mix.{s}": (H * d, width) for s in "rkvg"})
            new.update({"mix.w1": (rank, width), "mix.w2": (H * d, rank), "mix.w0": (H * d,), "mix.u": (H, d), "mix.norm": (H * d,), "mix.o": (width, H * d)})
        else:
            v = m["vdim"]
            new.update({"mix.q": (H * d, width), "mix.f": (H * d, width), "mix.f.b": (H * d,), "mix.lower": (H * d,), "mix.v": (H * v, width), "mix.norm": (v,),
                        "mix.o": (width, H * v)})
        shapes.update({p + n: s for n, s in new.items()})
    return _random_model(ctx, cfg, shapes, max_rows)


def nefipel_config(width):
    """Heads of 128 in groups of four, then two maps of 64 over values of 128; dense gated parts in every other layer, else 60
    experts and 4 identity experts, 8 of them a token, and a shared one: as many multiplications a token as a dense part has."""
    h = width // 128
    att = {"heads": h, "kv_heads": max(h // 4, 1), "dim": 128, "vdim": 128, "rot": {"base": 10000.0, "dims": 64}, "scale": 128 ** -0.5}
    yarn = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    diff = {"heads": h, "kv_heads": max(h // 4, 1), "dim": 64, "vdim": 128, "rot": {"base": 10000.0, "dims": 64, "scaling": yarn}, "scale": 0.125, "diff": 0.5}
    moe = {"kind": "moe", "expert": {"ff": width * 3 // 8}, "shared": {"ff": width * 9 // 8},
           "router": {"experts": 60, "identity": 4, "top": 8, "groups": {"count": 8, "keep": 4}}}
    block = [{"type": "attention", "mixer": att, "mlp": {"kind": "dense", "ff": width * 11 // 4}}, {"type": "attention_2", "mixer": diff, "mlp": moe}]
    return {"architecture": "Nefipel", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-6}, "postln_alpha": 2.5, "embedding": {"scale": 8.0},
            "layers": block * (LAYERS // 2)}


def random_nefipel(ctx, width, max_rows):
    cfg = nefipel_config(width)
    shapes = {"embed": (VOCAB, width), "final.norm": (width,)}
    for i, e in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", e["mixer"], e["mlp"]
        H, G, d, v, maps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], 2 if e["type"] == "attention_2" else 1
        new = {"norm1": (width,), "norm2": (width,), "mix.q": (H * maps * d, width), "mix.k": (G * maps * d, width), "mix.v": (G * v, width),
               "mix.o": (width, H * v), "mix.q.norm": (d,), "mix.k.norm": (d,)}
        if maps == 1:
            new.update({"mix.q.b": (H * d,), "mix.k.b": (G * d,), "mix.v.b": (G * v,), "mix.g": (H * v, width)})
        else:
            new.update({"mix." + n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")})
        if mlp["kind"] == "dense":
            new.update({"mlp.gate": (mlp["ff"], width), "mlp.up": (mlp["ff"], width), "mlp.down": (width, mlp["ff"])})
        else:
            n, f, s = mlp["router"]["experts"], mlp["expert"]["ff"], mlp["shared"]["ff"]
            new.update({"mlp.router": (n + mlp["router"]["identity"], width), "mlp.correction": (n + mlp["router"]["identity"],), "mlp.shared.sg": (1, width),
                        "mlp.shared.up": (s, width), "mlp.shared.down": (width, s)})
            for k in range(n):
                new.update({f"mlp.e{k}.up": (f, width), f"mlp.e{k}.down": (width, f)})
        shapes.update({p + n: s for n, s in new.items()})
    return _random_model(ctx, cfg, shapes, max_rows)


def lipelix_config(width):
    """Attention over everything, attention in a window of 512 with 16 kept tokens (heads of 128 in groups of four), generalised
    delta rule with heads of 128; the gates of the results are taken off the feed-forward parts, so a layer is as large as Zusepel's."""
    h, mlp = width // 128, {"kind": "dense", "ff": width * 25 // 8}
    att = {"heads": h, "kv_heads": max(h // 4, 1), "dim": 128, "vdim": 128, "rot": {"base": 10000.0, "dims": 128}, "scale": 128 ** -0.5, "v_mix": True}
    block = [("attention", att), ("attention_2", {**att, "mask": {"size": 512, "keep_first": 16}}), ("general_delta", {"heads": h, "dim": 128})]
    return {"architecture": "Lipelix", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-6}, "residual_mult": 0.5, "embedding": {"scale": 8.0},
            "layers": [{"type": t, "mixer": m, "mlp": mlp} for t, m in block * (LAYERS // 3)]}


def random_lipelix(ctx, width, max_rows, rank=64):
    cfg = lipelix_config(width)
    shapes = {"embed": (VOCAB, width), "head": (VOCAB, width), "final.norm": (width,)}
    for i, e in enumerate(cfg["layers"]):
        p, m, ff = f"l{i}.", e["mixer"], e["mlp"]["ff"]
        new = {n: (width,) for n in ("norm1", "norm1b", "norm2", "norm2b", "shift", "rg1.b", "rg2.b")}
        new.update({"rg1": (width, width), "rg2": (width, width), "mlp.up": (ff, width), "mlp.down": (width, ff)})
        H, d = m["heads"], m["dim"]
        if e["type"] == "general_delta":
            new.update({f"mix.{s}": (H * d, width) for s in "rkvga"})
            new.update({"mix.a.b": (H * d,), "mix.w0": (H * d,), "mix.norm": (H * d,), "mix.w1": (rank, width), "mix.w2": (H * d, rank), "mix.o": (width, H * d)})
        else:
            G, v = m["kv_heads"], m["vdim"]
            new.update({"mix.q": (H * d, width), "mix.k": (G * d, width), "mix.v": (G * v, width), "mix.o": (width, H * v), "mix.vmix": (1,)})
            if e["type"] == "attention":
                new.update({"mix.q.norm": (H * d,), "mix.k.norm": (G * d,), "mix.sink": (H,)})
        shapes.update({p + n: s for n, s in new.items()})
    return _random_model(ctx, cfg, shapes, max_rows)


def random_gpt(ctx, width, max_rows):
    """The fixed-block model of the same width, depth, feed-forward size and vocabulary (head size 16, its tuned case)."""
    ff, L = width * 11 // 4, LAYERS
    m = GPTModel(ctx, VOCAB, MAX_POS, width, width // 16, L, ff, maxRows=max_rows)
    noise = np.random.default_rng(0).standard_normal(VOCAB * width, dtype=np.float32) * np.float32(width ** -0.5)
    sizes = [VOCAB * width, MAX_POS * width]
    for _ in range(L):
        sizes += [width * width] * 4 + [width * ff] * 3 + [width] * 2
    sizes += [width, VOCAB * width]
    m.setParameters([np.ones(n, np.float32) if n == width else np.resize(noise, n) for n in sizes])
    return m


def _decode(ctx, model, batch, ctx_len, steps):
    pool = model.newPool(batch * -(-(ctx_len + steps + 8) // 16), batch)
    rng = np.random.default_rng(1)
    seqs = [pool.seq_alloc() for _ in range(batch)]
    toks, per = np.zeros(batch, np.int32), max(1, model.maxRows // ctx_len)
    for i in range(0, batch, per):
        ps = [rng.integers(1, VOCAB, ctx_len).astype(np.int32) for _ in seqs[i:i + per]]
        if isinstance(model, GPTModel):
            _, toks[i:i + per] = model.forwardPrefillBatch(pool, seqs[i:i + per], ps)
        else:
            ends = np.cumsum([len(p) for p in ps]) - 1
            _, toks[i:i + per] = model.step(pool, seqs[i:i + per], ps, ends, want_logits=False, want_next=True)
    lens, ids, ms = np.full(batch, ctx_len, np.int32), np.asarray(seqs, np.int32), []
    for i in range(steps):
        t0 = time.perf_counter()
        _, toks = model.forwardDecodeBatch(pool, ids, toks, lens, lens, want_logits=False)
        if i >= 4:
            ms.append((time.perf_counter() - t0) * 1e3)
        lens += 1
    pool.close()
    return float(np.median(ms))


def _prefill(ctx, model, batch, seq_len, repeats):
    pool = model.newPool(batch * -(-seq_len // 16), batch)
    rng = np.random.default_rng(2)
    ps = [rng.integers(1, VOCAB, seq_len).astype(np.int32) for _ in range(batch)]
    seqs, best = [pool.seq_alloc() for _ in range(batch)], []
    e0, e1 = Event(ctx), Event(ctx)
    for i in range(repeats + 2):
        for s in seqs:
            pool.clear(s, zero_fill=False)
        ctx.synchronize()
        e0.record()
        if isinstance(model, GPTModel):
            model.forwardPrefillBatch(pool, seqs, ps)
        else:
            model.step(pool, seqs, ps, np.arange(1, batch + 1) * seq_len - 1, want_logits=False, want_next=True)
        e1.record()
        if i >= 2:
            best.append(e0.elapsed_ms(e1))
    pool.close()
    return float(np.median(best))


def run_decoder(ctx, widths=(1024, 2048), batches=(1, 16, 64), prompts=((1, 2048), (8, 1024)), ctx_len=1500, steps=24, repeats=5, models=("lipelix", "nefipel", "zusepel", "somopel", "gpt")):
    out = {"workload": f"{LAYERS} layers, vocabulary {VOCAB}, random weights; prefill = prompts of one call, decode at context {ctx_len}+",
           "timing": "prefill: CUDA events around the call; decode: host clock around a step that reads its ids back; medians", "sizes": []}
    for w in widths:
        row = {"width": w}
        for name, make in (("lipelix", random_lipelix), ("nefipel", random_nefipel), ("zusepel", random_zusepel), ("somopel", random_somopel), ("gpt", random_gpt)):
            if name not in models:
                continue
            m = make(ctx, w, 8192)
            r = {}
            for b, n in prompts:
                ms = _prefill(ctx, m, b, n, repeats)
                r[f"prefill_{b}x{n}"] = {"ms": ms, "tokens_per_s": b * n / ms * 1e3}
            for b in batches:
                ms = _decode(ctx, m, b, ctx_len, steps)
                r[f"decode_b{b}"] = {"ms": ms, "tokens_per_s": b / ms * 1e3}
            row[name] = r
            m.close()
        out["sizes"].append(row)
    return out
