// Kernels of the layered decoder (decoder.cu): embedding and layer norm, paged attention over key heads of any size, and
// the recurrent mixers.  AT is the activation (and cache) type: __nv_bfloat16 when serving, float in the exact mode.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace jgpt {
namespace mix {

// One entry of a step: T consecutive tokens of a sequence, rows [row0, row0 + T) of the packed activations, first token at
// position pos0.  conv_set: which of the two copies of the convolution history holds the inputs before pos0.
struct Seg {
    int seq, row0, T, pos0, conv_set, pad;
};

// What a step brings, on the device.
struct StepDesc {
    const int *tok, *pos, *seq;  // per row
    const Seg *segs;
    const int2 *tiles;           // (entry, first token) of every query tile of the entries with more than one token
    const int *singles;          // entries with one token
    const int *short_segs;       // entries whose recurrences run token by token
    const int2 *long_segs;       // the others: (entry, index of its first chunk)
    const int2 *chunks;          // (entry, first token) of the long entries' chunks of kRecChunk tokens
    const int *want;             // rows whose logits are wanted
    int rows, n_segs, n_tiles, n_singles, n_short, n_long, n_chunks, n_want;
    int qt;                      // tokens per query tile
    int max_len;                 // upper bound of pos0 + T (sizes the split of single-token attention)
};

// ---- norm.cu ---------------------------------------------------------------------------------------
// x[r] = LN(embed[tok[r]] * scale + pos_table[pos[r]]) (norm applied when gamma is set), h[r] = LN(x[r]; next norm).
// Rows are W wide, h has row stride ldh (elements past W are zeroed).
struct NormW {
    const float *gamma, *beta;
};
int32_t launch_embed(bool f32, const StepDesc &d, const void *embed, int ld_embed, const void *pos_table, int ld_pos, float scale,
                     NormW embed_norm, NormW next, float eps, float *x, void *h, int W, int ldh, int vocab, int max_pos, int *status, int pdl,
                     cudaStream_t st);
int32_t launch_layer_norm(bool f32, const float *x, const int *rowsel, NormW w, float eps, void *h, int rows, int W, int ldh, int pdl,
                          cudaStream_t st);

// ---- attn_gqa.cu -----------------------------------------------------------------------------------
struct AttnArgs {
    const void *proj;   // [rows, ldp] projections of the layer
    int ldp, q_off, k_off, v_off, g_off;  // column offsets; g_off < 0: no output gate
    int heads, kv_heads, D;  // query heads, key heads, padded head size (q, k and v alike)
    int chunk;          // a query sees the keys of its own chunk of this many positions (0: all earlier positions)
    float scale, out_scale;
    void *kv;           // this layer's pages: [block][kv head][K 16 x D | V 16 x D]
    const int *table;
    int n_blocks, mbs;
    void *out;          // [rows, ldo], head h at out_off + h * D
    int ldo, out_off;
    int sm_count;
    int *status;
};
int32_t launch_attention(bool f32, const StepDesc &d, const AttnArgs &a, int pdl, cudaStream_t st);
int attn_padded_head(int dim, int vdim);          // 0: not supported
int attn_query_tile(int heads, int kv_heads);     // tokens per query tile of the multi-token kernel

// ---- recurrent.cu ----------------------------------------------------------------------------------
enum RecKind : int { REC_GLA = 0, REC_DELTA = 1 };
struct RecArgs {
    int kind;
    const void *proj;   // [rows, ldp]
    int ldp, q_off, k_off, v_off, b_off, g_off;  // b: step-size column (delta); g: output gate inside proj (GLA)
    const void *z;      // [rows, ldz]: decay logits at z_off, output gate at zg_off (delta)
    int ldz, z_off, zg_off;
    int heads, kv_heads, DK, DV;  // padded head sizes
    int dim, vdim;      // true head sizes
    float tau, out_scale, eps;
    const float *conv_q, *conv_k, *conv_v;  // [channels][taps] (padded channels), taps = 0: no convolution
    int taps;
    const float *decay_bias;  // [heads * DK]
    const float *a_log;       // [heads] (delta)
    const float *norm_w;      // [DV]
    uint8_t *state;     // of sequence slot 0, this layer's part
    uint64_t state_stride;    // bytes between sequence slots
    uint64_t conv_off;  // byte offset of the convolution history [2][taps - 1][channels] inside the part
    int max_seqs;
    void *out;          // [rows, ldo]
    int ldo, out_off;
    float *raw;         // [rows, heads * DV] scratch for heads whose columns are cut over several CTAs
    float *chunk_ws;    // records of the chunked form
    uint64_t chunk_ws_floats;
    int sm_count;
    int *status;
};
constexpr int kRecChunk = 16;
int rec_chunk_min_tokens(bool f32);  // entries of at least this many tokens take the chunked form (0: none)
uint64_t rec_chunk_record_floats(int kind, int DK, int DV);
int32_t launch_recurrent_chunks(bool f32, const StepDesc &d, const RecArgs &a, int pdl, cudaStream_t st);
int32_t launch_recurrent(bool f32, const StepDesc &d, const RecArgs &a, int pdl, cudaStream_t st);
int rec_padded_key(int dim);    // 0: not supported
int rec_padded_value(int vdim);
uint64_t rec_state_bytes(const RecArgs &a, int elem_bytes, uint64_t *conv_off);

}  // namespace mix
}  // namespace jgpt
