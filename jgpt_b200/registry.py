"""Model registry: config.json's "architecture" picks the design, the design describes the model.

A design is a function ``(config, shape_of) -> DecoderConfig``; ``shape_of(name)`` gives the shape of a tensor of the
weight file for sizes that only the tensors hold.
"""
from __future__ import annotations

import json
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


# ---- Somopel -------------------------------------------------------------------------------------------
def _norm(names, role, name):
    names[role], names[role + 1] = name, name + ".b"


def _attention(m, p, shape_of, out_scale):
    return D.Mixer(D.MIX_ATTENTION, m["heads"], m["kv_heads"], m["dim"], m["vdim"], chunk=m["mask"]["size"], gate=True,
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
