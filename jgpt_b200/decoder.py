"""Layered decoders: models the library assembles from layer descriptions (``jgpt_decoder_create``).

``DecoderConfig`` is the description (what ``jgpt_layer_spec`` holds) plus the names of the tensors each part is loaded
from; designs build it from their config.json (``registry.py``).  ``DecoderModel`` has the methods of ``GPTModel`` that do
not depend on its fixed block, so generation and ``ContinuousBatcher`` take either.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

import numpy as np

from . import binding as B
from .kv_cache import KvPool
from .runtime import Context

MIX_ATTENTION, MIX_GLA, MIX_DELTA, MIX_HGRN2, MIX_WKV, MIX_LATENT, MIX_GENERAL_DELTA = range(1, 8)
NORM_LAYER, NORM_RMS = 0, 1
FF_GATED_GELU, FF_XIELU, FF_GATED_RELU, FF_MOE, FF_RELU2 = range(5)
ACT_RELU, ACT_RELU2, ACT_GELU_TANH = range(3)
GATE_NONE, GATE_HEAD, GATE_ELEMENT = range(3)
QK_NORM_NONE, QK_NORM_HEAD, QK_NORM_ALL, QK_NORM_UNIT = range(4)
SINK_NONE, SINK_LEARNED, SINK_ZERO = range(3)
NO_LIMIT = 1 << 30  # positions of a model without a table of them
DTYPES = {"bfloat16": 0, "float32": 1}
BLOCK_TOKENS = 16
MAX_BRANCHES = 2


class _MixerSpec(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("kind", "heads", "kv_heads", "dim", "vdim", "chunk", "gate", "taps", "rank_a", "rank_g")] + \
               [(n, C.c_float) for n in ("score_scale", "tau", "out_scale")] + \
               [(n, C.c_int32) for n in ("window", "q_rank", "kv_rank", "rot_dim", "rot_dims", "kv_from")] + \
               [(n, C.c_double) for n in ("rot_base", "rot_factor", "rot_original", "rot_fast", "rot_slow")] + \
               [(n, C.c_int32) for n in ("rot_interleaved", "qkv_bias", "qk_norm", "maps")] + [("diff", C.c_float)] + \
               [(n, C.c_int32) for n in ("keep", "sink", "v_mix")] + [("decay_rate", C.c_float)]


class _MoeSpec(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("experts", "identity", "top", "groups", "keep", "ff", "shared_ff", "act", "shared_act")]


class _LayerSpec(C.Structure):
    _fields_ = [("n_branches", C.c_int32), ("branch", _MixerSpec * MAX_BRANCHES), ("ff", C.c_int32), ("ff_kind", C.c_int32), ("moe", _MoeSpec)]


class _DecoderSpec(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("vocab", "width", "max_positions", "n_layers", "embed_norm", "pos_table", "norm", "head", "layer_scale",
                                           "depth_average")] + \
               [(n, C.c_float) for n in ("eps", "embed_scale", "logit_scale", "residual_mult")] + \
               [("norm_after", C.c_int32), ("residual_scale", C.c_float)] + [(n, C.c_int32) for n in ("norm_both", "token_shift", "residual_gate")]


# tensor roles (JGPT_W_* of the header)
W_EMBED, W_POS, W_EMBED_NORM, W_EMBED_NORM_B, W_FINAL_NORM, W_FINAL_NORM_B, W_HEAD = range(7)
W_NORM1, W_NORM1_B, W_NORM2, W_NORM2_B, W_FF_GATE, W_FF_UP, W_FF_DOWN, W_LS1, W_LS2, W_DWA = range(10, 20)
(W_Q, W_K, W_V, W_O, W_G, W_B, W_A1, W_A2, W_DECAY_BIAS, W_A_LOG, W_G1, W_G2, W_HEAD_NORM, W_CONV_Q, W_CONV_K,
 W_CONV_V, W_MU_R, W_MU_K, W_MU_V, W_MU_G, W_MU_W, W_BONUS, W_LOWER, W_F, W_DQ, W_DQ_NORM, W_UQ, W_DKV, W_DKV_NORM, W_UK, W_UV,
 W_FF_ACT, W_Q_BIAS, W_K_BIAS, W_V_BIAS, W_Q_NORM, W_K_NORM, W_LQ1, W_LK1, W_LQ2, W_LK2, W_SINK,
 W_VMIX, W_B_BIAS) = range(20, 64)
W_ROUTER, W_CORRECTION, W_SHARED_GATE, W_SHARED_UP, W_SHARED_DOWN, W_EXPERT_UP, W_EXPERT_DOWN = range(64, 71)
W_POST1, W_POST2, W_SHIFT, W_RG1, W_RG1_B, W_RG2, W_RG2_B = range(80, 87)


@dataclass
class Mixer:
    kind: int
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    chunk: int = 0
    gate: int = GATE_NONE
    taps: int = 0
    rank_a: int = 0
    rank_g: int = 0
    score_scale: float = 1.0
    tau: float = 1.0
    out_scale: float = 1.0
    window: int = 0
    q_rank: int = 0
    kv_rank: int = 0
    rot_dim: int = 0
    rot_dims: int = 0
    kv_from: int = 0  # 1 + the layer whose latent cache is read, 0: its own
    rot_base: float = 0.0
    rot_factor: float = 0.0
    rot_original: float = 0.0
    rot_fast: float = 0.0
    rot_slow: float = 0.0
    rot_interleaved: bool = False
    qkv_bias: bool = False
    qk_norm: int = QK_NORM_NONE
    maps: int = 1  # 2: differential, the second map's output times lambda is taken off the first one's
    diff: float = 0.0
    keep: int = 0
    sink: int = SINK_NONE
    v_mix: bool = False
    decay_rate: float = 1.0
    tensors: dict = field(default_factory=dict)  # role -> tensor name


@dataclass
class Moe:
    """Experts W_down act(W_up h): the last ``identity`` router outputs hand h on, a shared expert runs for every token."""
    experts: int
    top: int
    ff: int
    identity: int = 0
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0
    act: int = ACT_RELU2
    shared_act: int = ACT_RELU2
    tensors: list = field(default_factory=list)  # per expert: role -> tensor name


@dataclass
class Layer:
    branches: list
    ff: int = 0
    tensors: dict = field(default_factory=dict)
    ff_kind: int = FF_GATED_GELU
    moe: Moe | None = None


@dataclass
class DecoderConfig:
    vocab: int
    width: int
    max_positions: int
    eps: float
    layers: list
    embed_norm: bool = False
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    pos_table: bool = True
    norm: int = NORM_LAYER
    head: bool = False
    layer_scale: bool = False
    depth_average: bool = False
    residual_mult: float = 1.0
    norm_after: bool = False
    residual_scale: float = 1.0
    norm_both: bool = False
    token_shift: bool = False
    residual_gate: bool = False
    tensors: dict = field(default_factory=dict)

    def all_tensors(self):
        """(layer, branch, role, name) of every tensor the model needs."""
        for role, name in self.tensors.items():
            yield -1, -1, role, name
        for i, layer in enumerate(self.layers):
            for role, name in layer.tensors.items():
                yield i, -1, role, name
            for j, m in enumerate(layer.branches):
                for role, name in m.tensors.items():
                    yield i, j, role, name
            for e, names in enumerate(layer.moe.tensors if layer.moe else ()):
                for role, name in names.items():
                    yield i, MAX_BRANCHES + e, role, name


class DecoderModel:
    def __init__(self, ctx: Context, config: DecoderConfig, dtype="bfloat16", maxRows=2048):
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype}: one of {', '.join(DTYPES)}")
        self.ctx, self._lib, self.config, self.dtype = ctx, ctx._lib, config, dtype
        self.vocabSize, self.maxSeqLen, self.dModel = config.vocab, config.max_positions, config.width
        self.numLayers, self.maxRows = len(config.layers), maxRows
        layers = (_LayerSpec * len(config.layers))()
        for spec, layer in zip(layers, config.layers):
            if not 1 <= len(layer.branches) <= 2:
                raise ValueError(f"a layer has one or two mixer branches, not {len(layer.branches)}")
            spec.n_branches, spec.ff, spec.ff_kind = len(layer.branches), layer.ff, layer.ff_kind
            for b, m in zip(spec.branch, layer.branches):
                for n, t in _MixerSpec._fields_:
                    setattr(b, n, int(getattr(m, n)) if t is C.c_int32 else getattr(m, n))
            if layer.moe:
                for n, _ in _MoeSpec._fields_:
                    setattr(spec.moe, n, getattr(layer.moe, n))
        top = _DecoderSpec(n_layers=len(config.layers))
        for n, t in _DecoderSpec._fields_:
            if n != "n_layers":
                setattr(top, n, int(getattr(config, n)) if t is C.c_int32 else getattr(config, n))
        h = C.c_uint64()
        B.check(self._lib.jgpt_decoder_create(ctx.handle, C.byref(top), layers, DTYPES[dtype], maxRows, C.byref(h)))
        self.handle = h.value

    # ---- weights -------------------------------------------------------------------------------
    def setTensor(self, layer, branch, role, array):
        a = np.ascontiguousarray(array, np.float32)
        rows, cols = (1, a.size) if a.ndim == 1 else a.shape
        B.check(self._lib.jgpt_decoder_set_tensor(self.handle, layer, branch, role, a.ctypes.data, rows, cols))

    def loadTensors(self, get):
        """``get(name)`` returns the array of a tensor name of the configuration."""
        for layer, branch, role, name in self.config.all_tensors():
            try:
                self.setTensor(layer, branch, role, get(name))
            except ValueError as e:
                raise ValueError(f"{name}: {e}") from None

    def newPool(self, n_blocks, max_seqs, max_blocks_per_seq=None) -> "DecoderPool":
        return DecoderPool(self, n_blocks, max_seqs, max_blocks_per_seq or min(n_blocks, -(-self.maxSeqLen // BLOCK_TOKENS)))

    # ---- forward step --------------------------------------------------------------------------
    def step(self, pool: KvPool, seqs, tokens, want=(), want_logits=True, want_next=False):
        """One mixed step: ``tokens[i]`` continues sequence ``seqs[i]``; ``want`` = rows of the concatenated tokens.
        Returns (logits [len(want), vocab] or None, greedy next tokens [len(want)] or None)."""
        starts = np.zeros(len(seqs) + 1, np.int32)
        starts[1:] = np.cumsum([len(t) for t in tokens])
        ids = np.ascontiguousarray(np.concatenate([np.asarray(t, np.int32) for t in tokens]), np.int32)
        sq, w = np.ascontiguousarray(seqs, np.int32), np.ascontiguousarray(want, np.int32)
        logits = np.empty((w.size, self.vocabSize), np.float32) if want_logits else None
        nxt = np.empty(w.size, np.int32) if want_next else None
        B.check(self._lib.jgpt_forward_step(self.handle, pool.handle, sq.size, sq.ctypes.data, starts.ctypes.data, ids.ctypes.data, w.size,
                                            w.ctypes.data if w.size else None, logits.ctypes.data if logits is not None else None,
                                            nxt.ctypes.data if nxt is not None else None))
        return logits, nxt

    def captureLayers(self, rows) -> np.ndarray:
        """The residual after every layer of the next step lands in the returned array, [layers, rows, width]."""
        out = np.empty((self.numLayers, rows, self.dModel), np.float32)
        B.check(self._lib.jgpt_decoder_capture_layers(self.handle, out.ctypes.data, out.size))
        return out

    def forwardDecodeBatch(self, pool, seqs, tokens, cacheLenBefore, ropePositions=None, want_logits=True):
        """One decode step for n independent sequences -> (logits [n, vocab] or None, greedy next tokens [n])."""
        sq, tk, lb = (np.ascontiguousarray(x, np.int32) for x in (seqs, tokens, cacheLenBefore))
        rp = lb if ropePositions is None else np.ascontiguousarray(ropePositions, np.int32)
        logits = np.empty((sq.size, self.vocabSize), np.float32) if want_logits else None
        nxt = np.empty(sq.size, np.int32)
        B.check(self._lib.jgpt_forward_decode(self.handle, pool.handle, sq.ctypes.data, tk.ctypes.data, lb.ctypes.data, rp.ctypes.data, sq.size,
                                              logits.ctypes.data if want_logits else None, nxt.ctypes.data))
        return logits, nxt

    def forwardDecodeSampleBatch(self, pool, seqs, tokens, cacheLenBefore, temperature, topK, u01):
        """One decode step + ``sampleNextToken`` per row on the device with the uniform draws ``u01`` -> next tokens [n]."""
        sq, tk, lb = (np.ascontiguousarray(x, np.int32) for x in (seqs, tokens, cacheLenBefore))
        u = np.ascontiguousarray(u01, np.float32)
        if u.size != sq.size:
            raise ValueError("one uniform draw per row")
        nxt = np.empty(sq.size, np.int32)
        B.check(self._lib.jgpt_forward_decode_sample(self.handle, pool.handle, sq.ctypes.data, tk.ctypes.data, lb.ctypes.data, lb.ctypes.data,
                                                     sq.size, float(temperature), int(topK), u.ctypes.data, nxt.ctypes.data))
        return nxt

    # ---- generation ----------------------------------------------------------------------------
    def generateGpuKv(self, inputTokens, maxNewTokens, temperature=0.0, topK=0, pool: KvPool | None = None, rng=None):
        """Ids [S + maxNewTokens]: the prompt, then the picked tokens, a zero tail after an early stop on id 0 (the rules of
        ``GPTModel.generateGpuKv``; no sliding window: prompt and new tokens must fit the model's positions)."""
        prompt = np.ascontiguousarray(inputTokens, np.int32).reshape(-1)
        own = pool is None
        if own:
            pool = self.newPool(-(-min(self.maxSeqLen, prompt.size + maxNewTokens) // BLOCK_TOKENS), 1)
        try:
            out = np.zeros(prompt.size + maxNewTokens, np.int32)
            if temperature <= 0:
                n = C.c_int32()
                B.check(self._lib.jgpt_generate_greedy(self.handle, pool.handle, prompt.ctypes.data, prompt.size, maxNewTokens,
                                                       out.ctypes.data, C.byref(n)))
                return out
            rng = rng or np.random.default_rng()
            out[: prompt.size] = prompt
            seq = pool.seq_alloc()
            try:
                for t0 in range(0, prompt.size - 1, self.maxRows):  # all but the last prompt token, in portions
                    self.step(pool, [seq], [prompt[t0:min(t0 + self.maxRows, prompt.size - 1)]], want_logits=False)
                for j in range(maxNewTokens):
                    at = prompt.size + j
                    tok = self.forwardDecodeSampleBatch(pool, [seq], [out[at - 1]], [at - 1], temperature, topK, [rng.random()])[0]
                    out[at] = tok
                    if tok == 0:
                        break
            finally:
                pool.seq_free(seq)
            return out
        finally:
            if own:
                pool.close()

    def close(self):
        if self.handle:
            self._lib.jgpt_model_destroy(self.handle)
            self.handle = 0


class DecoderPool(KvPool):
    """The paged store of a layered decoder: the allocator of ``KvPool`` over pages of the model's own geometry, plus a
    slot of recurrent state per sequence."""

    def __init__(self, model: DecoderModel, n_blocks, max_seqs, max_blocks_per_seq):
        self.ctx, self._lib = model.ctx, model._lib
        self.n_blocks, self.max_seqs, self.max_blocks_per_seq = n_blocks, max_seqs, max_blocks_per_seq
        self.max_positions = max_blocks_per_seq * BLOCK_TOKENS
        h = C.c_uint64()
        B.check(self._lib.jgpt_decoder_new_pool(model.handle, n_blocks, max_seqs, max_blocks_per_seq, C.byref(h)))
        self.handle = h.value
