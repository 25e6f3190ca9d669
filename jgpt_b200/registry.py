"""Model registry: config.json's "architecture" picks the design, the design describes the model.

A design is a function ``(config, shape_of) -> DecoderConfig``; ``shape_of(name)`` gives the shape of a tensor of the
weight file for sizes that only the tensors hold.
"""
from __future__ import annotations

import json
import math
import os

from . import decoder as D
from .safetensors import SafetensorsFile

DESIGNS = {}


def register(name):
    def add(fn):
        DESIGNS[name] = fn
        return fn
    return add


def describe(config: dict, shape_of) -> D.DecoderConfig:
    name = config.get("architecture")
    if name not in DESIGNS:
        raise ValueError(f"architecture {name!r} is not registered (known: {', '.join(sorted(DESIGNS))})")
    return DESIGNS[name](config, shape_of)


def load_model(ctx, folder, dtype="bfloat16", max_rows=2048) -> D.DecoderModel:
    """The model of a folder with config.json and model.safetensors, its weights on the device."""
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    w = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    try:
        model = D.DecoderModel(ctx, describe(config, w.shape), dtype, max_rows)
        try:
            model.loadTensors(w.get)
        except Exception:
            model.close()
            raise
        return model
    finally:
        w.close()


def _rotation(rot):
    yarn = rot.get("scaling")
    return {"rot_dims": rot["dims"], "rot_base": rot["base"],
            **({"rot_" + k: yarn[k] for k in ("factor", "original", "fast", "slow")} if yarn else {})}


# ---- Somopel -------------------------------------------------------------------------------------------
def _norm(names, role, name):
    names[role], names[role + 1] = name, name + ".b"


def _attention(m, p, shape_of, out_scale):
    return D.Mixer(D.MIX_ATTENTION, m["heads"], m["kv_heads"], m["dim"], m["vdim"], chunk=m["mask"]["size"], gate=D.GATE_HEAD,
                   score_scale=m["scale"], out_scale=out_scale,
                   tensors={D.W_Q: p + "q", D.W_K: p + "k", D.W_V: p + "v", D.W_G: p + "g", D.W_O: p + "o"})


def _gla(m, p, shape_of, out_scale):
    return D.Mixer(D.MIX_GLA, m["heads"], m["heads"], m["dim"], m["vdim"], rank_a=shape_of(p + "a1")[0], tau=m["tau"], out_scale=out_scale,
                   tensors={D.W_Q: p + "q", D.W_K: p + "k", D.W_V: p + "v", D.W_G: p + "g", D.W_O: p + "o", D.W_A1: p + "a1",
                            D.W_A2: p + "a2", D.W_DECAY_BIAS: p + "a2.b", D.W_HEAD_NORM: p + "norm"})


def _delta(m, p, shape_of):
    return D.Mixer(D.MIX_DELTA, m["heads"], m["kv_heads"], m["dim"], m["vdim"], taps=m["conv"], rank_a=shape_of(p + "a1")[0],
                   rank_g=shape_of(p + "g1")[0],
                   tensors={D.W_Q: p + "q", D.W_K: p + "k", D.W_V: p + "v", D.W_O: p + "o", D.W_B: p + "b", D.W_A1: p + "a1", D.W_A2: p + "a2",
                            D.W_DECAY_BIAS: p + "dt_bias", D.W_A_LOG: p + "A_log", D.W_G1: p + "g1", D.W_G2: p + "g2",
                            D.W_HEAD_NORM: p + "norm", D.W_CONV_Q: p + "q.conv", D.W_CONV_K: p + "k.conv", D.W_CONV_V: p + "v.conv"})


@register("Somopel")
def somopel(c, shape_of) -> D.DecoderConfig:
    """Layers of two kinds: 'parallel' (chunked softmax attention beside gated linear attention) and 'channel_delta'
    (gated delta rule with a decay per key channel); learned positions, tied logits."""
    layers = []
    for i, e in enumerate(c["layers"]):
        p, m, mlp = f"l{i}.", e["mixer"], e["mlp"]
        names = {}
        _norm(names, D.W_NORM1, p + "norm1")
        if e["type"] == "parallel":
            branches = [_attention(m["left"], p + "mix.left.", shape_of, m["left_scale"]), _gla(m["right"], p + "mix.right.", shape_of, m["right_scale"])]
        elif e["type"] == "channel_delta":
            branches = [_delta(m, p + "mix.", shape_of)]
        else:
            raise ValueError(f"layer {i}: mixer type {e['type']!r}")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
            _norm(names, D.W_NORM2, p + "norm2")
            names.update({D.W_FF_GATE: p + "mlp.gate", D.W_FF_UP: p + "mlp.up", D.W_FF_DOWN: p + "mlp.down"})
        layers.append(D.Layer(branches, mlp["ff"] if mlp else 0, names))
    names = {D.W_EMBED: "embed", D.W_POS: "pos"}
    _norm(names, D.W_EMBED_NORM, "embed.norm")
    _norm(names, D.W_FINAL_NORM, "final.norm")
    return D.DecoderConfig(c["vocab"], c["width"], c["max_positions"], c["norm"]["eps"], layers, embed_norm=True,
                           embed_scale=c["embedding"]["scale"], logit_scale=c["logit_scale"], tensors=names)


# ---- Zusepel -------------------------------------------------------------------------------------------
def _hgrn2(m, p):
    return D.Mixer(D.MIX_HGRN2, m["heads"], m["heads"], m["dim"], m["vdim"],
                   tensors={D.W_Q: p + "q", D.W_F: p + "f", D.W_DECAY_BIAS: p + "f.b", D.W_LOWER: p + "lower", D.W_V: p + "v", D.W_HEAD_NORM: p + "norm",
                            D.W_O: p + "o"})


def _wkv(m, p, shape_of):
    return D.Mixer(D.MIX_WKV, m["heads"], m["heads"], m["dim"], m["dim"], rank_a=shape_of(p + "w1")[0],
                   tensors={D.W_MU_R: p + "mu.r", D.W_MU_K: p + "mu.k", D.W_MU_V: p + "mu.v", D.W_MU_G: p + "mu.g", D.W_MU_W: p + "mu.w", D.W_Q: p + "r",
                            D.W_K: p + "k", D.W_V: p + "v", D.W_G: p + "g", D.W_A1: p + "w1", D.W_A2: p + "w2", D.W_DECAY_BIAS: p + "w0",
                            D.W_BONUS: p + "u", D.W_HEAD_NORM: p + "norm", D.W_O: p + "o"})


def _latent(m, p):
    names = {D.W_DQ: p + "dq", D.W_DQ_NORM: p + "dq.norm", D.W_UQ: p + "uq", D.W_UK: p + "uk", D.W_UV: p + "uv", D.W_O: p + "o"}
    shared = m.get("kv_from")
    if shared is None:
        names.update({D.W_DKV: p + "dkv", D.W_DKV_NORM: p + "dkv.norm"})
    return D.Mixer(D.MIX_LATENT, m["heads"], m["heads"], m["dim"], m["vdim"], window=(m.get("mask") or {}).get("size", 0), q_rank=m["q_rank"],
                   kv_rank=m["kv_rank"], rot_dim=m["rot_dim"], kv_from=0 if shared is None else 1 + shared, score_scale=m["scale"],
                   **_rotation(m["rot"]), tensors=names)


@register("Zusepel")
def zusepel(c, shape_of) -> D.DecoderConfig:
    """Layers of three kinds in any order: 'latent_attention' (sliding window, YaRN rotation, a layer may read an earlier
    layer's cache), 'wkv' and 'hgrn2' (recurrences); RMS norms, layer scales, averages over the depth, an xIELU feed-forward
    part, no table of positions."""
    layers = []
    for i, e in enumerate(c["layers"]):
        p, m, mlp = f"l{i}.", e["mixer"], e["mlp"]
        names = {D.W_NORM1: p + "norm1", D.W_LS1: p + "ls1", D.W_DWA: p + "dwa"}
        if e["type"] == "latent_attention":
            mixer = _latent(m, p + "mix.")
        elif e["type"] == "wkv":
            mixer = _wkv(m, p + "mix.", shape_of)
        elif e["type"] == "hgrn2":
            mixer = _hgrn2(m, p + "mix.")
        else:
            raise ValueError(f"layer {i}: mixer type {e['type']!r}")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
            names.update({D.W_NORM2: p + "norm2", D.W_LS2: p + "ls2", D.W_FF_UP: p + "mlp.up", D.W_FF_DOWN: p + "mlp.down", D.W_FF_ACT: p + "mlp.act"})
        layers.append(D.Layer([mixer], mlp["ff"] if mlp else 0, names, D.FF_XIELU))
    names = {D.W_EMBED: "embed", D.W_FINAL_NORM: "final.norm", D.W_HEAD: "head"}
    return D.DecoderConfig(c["vocab"], c["width"], D.NO_LIMIT, c["norm"]["eps"], layers, pos_table=False, norm=D.NORM_RMS, head=True, layer_scale=True,
                           depth_average=True, residual_mult=c["residual_mult"], tensors=names)


# ---- Nefipel -------------------------------------------------------------------------------------------
def _gated_heads(m, p):
    return D.Mixer(D.MIX_ATTENTION, m["heads"], m["kv_heads"], m["dim"], m["vdim"], gate=D.GATE_ELEMENT, score_scale=m["scale"], qkv_bias=True,
                   qk_norm=D.QK_NORM_HEAD, **_rotation(m["rot"]),
                   tensors={D.W_Q: p + "q", D.W_K: p + "k", D.W_V: p + "v", D.W_Q_BIAS: p + "q.b", D.W_K_BIAS: p + "k.b", D.W_V_BIAS: p + "v.b",
                            D.W_Q_NORM: p + "q.norm", D.W_K_NORM: p + "k.norm", D.W_G: p + "g", D.W_O: p + "o"})


def _differential(m, p):
    return D.Mixer(D.MIX_ATTENTION, m["heads"], m["kv_heads"], m["dim"], m["vdim"], score_scale=m["scale"], qk_norm=D.QK_NORM_HEAD, rot_interleaved=True,
                   maps=2, diff=m["diff"], **_rotation(m["rot"]),
                   tensors={D.W_Q: p + "q", D.W_K: p + "k", D.W_V: p + "v", D.W_Q_NORM: p + "q.norm", D.W_K_NORM: p + "k.norm", D.W_LQ1: p + "lq1",
                            D.W_LK1: p + "lk1", D.W_LQ2: p + "lq2", D.W_LK2: p + "lk2", D.W_O: p + "o"})


def _mixture(mlp, p, names):
    r, shared, groups = mlp["router"], mlp.get("shared"), mlp["router"].get("groups") or {}
    names.update({D.W_ROUTER: p + "router", D.W_CORRECTION: p + "correction"})
    if shared:
        names.update({D.W_SHARED_GATE: p + "shared.sg", D.W_SHARED_UP: p + "shared.up", D.W_SHARED_DOWN: p + "shared.down"})
    return D.Moe(r["experts"], r["top"], mlp["expert"]["ff"], identity=r.get("identity", 0), groups=groups.get("count", 1), keep=groups.get("keep", 1),
                 shared_ff=shared["ff"] if shared else 0,
                 tensors=[{D.W_EXPERT_UP: f"{p}e{e}.up", D.W_EXPERT_DOWN: f"{p}e{e}.down"} for e in range(r["experts"])])


@register("Nefipel")
def nefipel(c, shape_of) -> D.DecoderConfig:
    """Layers of two kinds in any order: 'attention' (normed, rotated heads with biases, a gate per element of the output) and
    'attention_2' (two maps per head, the second taken off the first); norms behind the sums; dense gated-relu parts and
    mixtures of experts with identity experts and a gated shared expert; tied logits."""
    layers = []
    for i, e in enumerate(c["layers"]):
        p, m, mlp = f"l{i}.", e["mixer"], e["mlp"]
        names, ff, kind, moe = {D.W_NORM1: p + "norm1"}, 0, D.FF_GATED_RELU, None
        if e["type"] == "attention":
            mixer = _gated_heads(m, p + "mix.")
        elif e["type"] == "attention_2":
            mixer = _differential(m, p + "mix.")
        else:
            raise ValueError(f"layer {i}: mixer type {e['type']!r}")
        if mlp is not None:
            names[D.W_NORM2] = p + "norm2"
            if mlp["kind"] == "dense":
                ff = mlp["ff"]
                names.update({D.W_FF_GATE: p + "mlp.gate", D.W_FF_UP: p + "mlp.up", D.W_FF_DOWN: p + "mlp.down"})
            elif mlp["kind"] == "moe":
                kind, ff, moe = D.FF_MOE, mlp["expert"]["ff"], _mixture(mlp, p + "mlp.", names)
            else:
                raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        layers.append(D.Layer([mixer], ff, names, kind, moe))
    return D.DecoderConfig(c["vocab"], c["width"], D.NO_LIMIT, c["norm"]["eps"], layers, pos_table=False, norm=D.NORM_RMS,
                           embed_scale=c["embedding"]["scale"], norm_after=True, residual_scale=c["postln_alpha"],
                           tensors={D.W_EMBED: "embed", D.W_FINAL_NORM: "final.norm"})


# ---- Lipelix -------------------------------------------------------------------------------------------
def _mixed_values(m, p, first):
    """The first layer that mixes its values is the one they come from: it has no share of its own."""
    if not m.get("v_mix"):
        return False, {}
    return True, {} if first else {D.W_VMIX: p + "vmix"}


def _normed_rows(m, p, v_mix, names):
    return D.Mixer(D.MIX_ATTENTION, m["heads"], m["kv_heads"], m["dim"], m["vdim"], score_scale=m["scale"], qk_norm=D.QK_NORM_ALL, sink=D.SINK_LEARNED,
                   v_mix=v_mix, **_rotation(m["rot"]),
                   tensors={D.W_Q: p + "q", D.W_K: p + "k", D.W_V: p + "v", D.W_Q_NORM: p + "q.norm", D.W_K_NORM: p + "k.norm", D.W_SINK: p + "sink",
                            D.W_O: p + "o", **names})


def _windowed(m, p, v_mix, names):
    return D.Mixer(D.MIX_ATTENTION, m["heads"], m["kv_heads"], m["dim"], m["vdim"], score_scale=m["scale"], qk_norm=D.QK_NORM_UNIT, sink=D.SINK_ZERO,
                   window=m["mask"]["size"], keep=m["mask"].get("keep_first", 0), v_mix=v_mix, **_rotation(m["rot"]),
                   tensors={D.W_Q: p + "q", D.W_K: p + "k", D.W_V: p + "v", D.W_O: p + "o", **names})


def _general_delta(m, p, shape_of):
    return D.Mixer(D.MIX_GENERAL_DELTA, m["heads"], m["heads"], m["dim"], m["dim"], rank_a=shape_of(p + "w1")[0], decay_rate=math.exp(-0.5),
                   tensors={D.W_Q: p + "r", D.W_K: p + "k", D.W_V: p + "v", D.W_G: p + "g", D.W_B: p + "a", D.W_B_BIAS: p + "a.b", D.W_A1: p + "w1",
                            D.W_A2: p + "w2", D.W_DECAY_BIAS: p + "w0", D.W_HEAD_NORM: p + "norm", D.W_O: p + "o"})


@register("Lipelix")
def lipelix(c, shape_of) -> D.DecoderConfig:
    """Layers of three kinds in any order: 'attention' (queries and keys normed as whole rows, all earlier positions, a learned
    sink), 'attention_2' (a sliding window with kept first tokens, unit heads, a sink of score 0) and 'general_delta' (recurrence);
    norms on both sides of every part, gated results, a token shift, values mixed with the first layer's."""
    layers, source = [], None
    for i, e in enumerate(c["layers"]):
        p, m, mlp = f"l{i}.", e["mixer"], e["mlp"]
        names = {D.W_NORM1: p + "norm1", D.W_POST1: p + "norm1b", D.W_SHIFT: p + "shift", D.W_RG1: p + "rg1", D.W_RG1_B: p + "rg1.b"}
        if e["type"] in ("attention", "attention_2"):
            v_mix, extra = _mixed_values(m, p + "mix.", source is None)
            source = i if source is None and v_mix else source
            mixer = (_normed_rows if e["type"] == "attention" else _windowed)(m, p + "mix.", v_mix, extra)
        elif e["type"] == "general_delta":
            mixer = _general_delta(m, p + "mix.", shape_of)
        else:
            raise ValueError(f"layer {i}: mixer type {e['type']!r}")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
            names.update({D.W_NORM2: p + "norm2", D.W_POST2: p + "norm2b", D.W_RG2: p + "rg2", D.W_RG2_B: p + "rg2.b", D.W_FF_UP: p + "mlp.up",
                          D.W_FF_DOWN: p + "mlp.down"})
        layers.append(D.Layer([mixer], mlp["ff"] if mlp else 0, names, D.FF_RELU2))
    return D.DecoderConfig(c["vocab"], c["width"], D.NO_LIMIT, c["norm"]["eps"], layers, pos_table=False, norm=D.NORM_RMS, head=True,
                           embed_scale=c["embedding"]["scale"], residual_mult=c["residual_mult"], norm_both=True, token_shift=True, residual_gate=True,
                           tensors={D.W_EMBED: "embed", D.W_FINAL_NORM: "final.norm", D.W_HEAD: "head"})
