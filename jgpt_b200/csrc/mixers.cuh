// Kernels of the layered decoder (decoder.cu): embedding and layer norm, paged attention over key heads of any size, and
// the recurrent mixers.  AT is the activation (and cache) type: __nv_bfloat16 when serving, float in the exact mode.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"
#include "gemm_nt.cuh"

namespace jgpt {
namespace mix {

// One entry of a step: T consecutive tokens of a sequence, rows [row0, row0 + T) of the packed activations, first token at
// position pos0.  conv_set: which of the two copies of the convolution history holds the inputs before pos0.
struct Seg {
    int seq, row0, T, pos0, conv_set, pad;
};

// What a step brings, on the device.
struct StepDesc {
    const int *tok, *pos, *seq, *ent;  // per row: token, position, sequence, entry
    const Seg *segs;
    const int2 *tiles;           // (entry, first token) of every query tile of the entries with more than one token
    const int *singles;          // entries with one token
    const int *short_segs;       // entries whose recurrences run token by token
    const int2 *long_segs;       // the others: (entry, index of its first chunk)
    const int2 *chunks;          // (entry, first token) of the long entries' chunks of kRecChunk tokens
    const int *want;             // rows whose logits are wanted
    const struct LatentEntry *lat_long;  // entries whose latent attention runs on written-out keys and values
    const int2 *lat_tiles;       // (index in lat_long, first token) of their query tiles
    const Seg *lat_singles, *lat_short;  // entries with one token; with more whose latent attention stays on the latents
    int rows, n_segs, n_tiles, n_singles, n_short, n_long, n_chunks, n_want, n_lat_short;
    int lat_short_max;           // tokens of the longest of the latter
    int lat_lo, lat_hi;          // rows from the first to the last of the entries that stay on the latents
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

// A row of the residual stream: the embedding of the row's token, or the weighted sum of the earlier layers' results
// (a plain residual is the sum over one slot without weights).
constexpr int kMaxRotations = 16;
struct Rotation {        // cos and sin of every row's angles, [rows][half] pairs, times mag
    const double *freq;
    float2 *out;
    int half;
    float mag;
};
struct RowSource {
    const void *embed;   // null: slots
    int ld_embed, vocab;
    float embed_scale;
    const float *slots, *weights;
    uint64_t slot_stride;
    int n_slots;
    Rotation rot[kMaxRotations];  // written beside the embedding
    int n_rot;
};
// Five mixes of a row with the one before it, h + (h' - h) mu_s; h' of an entry's first row comes from the sequence's state
// [2][W] (the copy conv_set names), its last row goes into the other copy.
struct ShiftArgs {
    const float *mu[5];  // null mu[0]: no mixes
    uint64_t out_stride; // elements between the mixes of h
    uint8_t *state;      // of slot 0, at the history
    uint64_t state_stride;
    int max_seqs;
};
// x[r] = source (when x is set), h[r] = x[r] / rms * gamma (x[r] itself without gamma), as mixes when sh has them; rowsel picks
// rows (null: all).
int32_t launch_residual_norm(bool f32, const StepDesc &d, const RowSource &src, const int *rowsel, int rows, const float *gamma, float eps, float *x,
                             void *h, const ShiftArgs &sh, int W, int ldh, int *status, int pdl, cudaStream_t st);

// The norm behind a sum: x[r] = S[r] / rms * gamma and h[r] = x[r], S = x itself, or with a mixture of experts
// S[r] = (alpha + weight of the identity experts) x[r] + sum of weight_s out[row of slot s] + shared gate * shared[r].
struct RouteSlot {
    int expert, rank;  // expert < 0: none; its row of the experts' products is offsets[expert] + rank
    float weight;
};
struct MoeSum {
    const void *out, *shared;  // [.., ld] activations; out null: no mixture; shared null: no shared expert
    int ld, top, cap;
    const RouteSlot *slots;    // [rows][top]
    const float2 *row_weights; // [rows]: identity experts, shared gate
    const int *offsets;
    float alpha;
};
int32_t launch_post_norm(bool f32, float *x, int rows, const float *gamma, float eps, void *h, const MoeSum &m, int W, int ldh, int pdl, cudaStream_t st);

// Between two parts with norms on either side: x[r] = source + mult * rms_norm(y[r] * sigmoid(gate[r])) * post, h[r] = rms_norm(x[r]) * pre,
// shifted[r] = h + (h' - h) share with h' as for ShiftArgs.  x, h, y and shifted have rows of ldw elements, zeros past W; weights likewise.
struct PartNorm {
    const float *x;            // residual so far; null: the embedding
    const void *y, *gate;      // y null: nothing is added; gate null: 1
    int ldg;
    const float *post;
    float mult;
    float *x_out;              // null: not stored
    const float *pre;
    void *h;                   // null: the residual only
    void *shifted;             // null: no token shift
    const float *share;
    uint8_t *state;            // of slot 0, at the row kept, [2][ldw]
    uint64_t state_stride;
    int max_seqs;
};
int32_t launch_part_norm(bool f32, const StepDesc &d, const RowSource &embed, const PartNorm &p, const int *rowsel, int rows, float eps, int W, int ldw,
                         int sm_count, int *status, int pdl, cudaStream_t st);

// ---- moe.cu ------------------------------------------------------------------------------------------
struct RouteArgs {
    const float *logits;       // [rows, ld]: experts, identity experts, the shared expert's gate (when shared is set)
    int ld, experts, identity, top, groups, keep, shared;
    const float *correction;   // [experts + identity]
    RouteSlot *slots;
    float2 *row_weights;
    int *list, *counts, *offsets, *ticket;  // rows of every expert [experts][cap]; counts and ticket are zero between launches
    int cap;
    nt::RowTile *tiles;
    int *n_tiles;
    int max_tiles, tile_rows;
};
int32_t launch_route(const RouteArgs &a, int rows, int pdl, cudaStream_t st);
// out[row of a tile] = the row of h that the tile's list names, ld bf16 elements each.
int32_t launch_moe_gather(const RouteArgs &a, const void *h, void *out, int ld, int pdl, cudaStream_t st);

// ---- attn_gqa.cu -----------------------------------------------------------------------------------
// Query heads in groups that share a key head.  Differential attention has two maps: a head's query and key are [map 1 | map 2],
// each map is an attention of its own over the same values, the second one's result times lambda is taken off the first one's
// and the difference brought to unit root mean square.  Padded sizes: DK per map, DV.
// Rows of a page are stored the way shared memory wants them: 16-byte pieces permuted by the row, or a row of an odd number of
// pieces, so that a page comes in as one bulk copy and eight rows are read without bank conflicts.
__host__ __device__ constexpr int page_row(int D) { return D % 64 == 0 ? D : D + 8; }
__host__ __device__ constexpr int page_chunk(int D, int row, int chunk) { return D % 64 == 0 ? chunk ^ (row & 7) : chunk; }
enum HeadGate : int { GATE_NONE = 0, GATE_HEAD = 1, GATE_ELEMENT = 2 };
struct AttnArgs {
    void *proj;         // [rows, ldp] projections of the layer
    int ldp, q_off, k_off, v_off, g_off;  // column offsets
    int heads, kv_heads, maps, DK, DV, dim, vdim;
    int gate;           // HeadGate: sigmoid of one column per head, or of a column per element of the output
    int window, keep;   // a query sees the last `window` positions and the first `keep` (window 0: as chunk says)
    int chunk;          // a query sees the keys of its own chunk of this many positions (0: all earlier positions)
    float scale, out_scale;
    const float *q_norm, *k_norm;  // weights [dim] of the RMS norm of every query and key head (map); null: none
    int whole_rows;     // the norm is that of all heads' rows at once, its weights padded [heads * DK]
    float2 *row_inv;    // [rows] 1 / root mean square of the query and key rows, written in steps with prompts
    float eps;
    const float *sink;  // [heads] score without a value; null: none
    const void *v_first;  // values become (1 - share) v + share v_first; null: no mixing
    int ld_first, vdim_first, DV_first;
    float v_share;
    const float2 *cs;   // [rows][half] cos and sin; the first 2 half elements of every head (map) turn; null: no rotation
    int half, interleaved;         // pairs (2 i, 2 i + 1), or (i, i + half)
    float lambda, diff_scale;
    void *kv;           // this layer's pages: [block][kv head][K 16 x page_row(maps DK) | V 16 x page_row(DV)]
    const int *table;
    int n_blocks, mbs;
    void *out;          // [rows, ldo], head h at out_off + h * DV
    int ldo, out_off;
    int sm_count;
    int *status;
    __host__ __device__ bool prepared() const { return q_norm || cs; }
    bool extra() const { return window > 0 || sink || whole_rows; }  // one map
    bool wide() const { return whole_rows || v_first; }  // a row's preparation needs more than its own heads  // heads are normed or rotated on their way
    __host__ __device__ int page_head() const { return kBlockTokens * (page_row(maps * DK) + page_row(DV)); }
};
int32_t launch_attention(bool f32, const StepDesc &d, const AttnArgs &a, int pdl, cudaStream_t st);
bool attn_padded_head(int dim, int vdim, int maps, int *DK, int *DV);  // false: not supported
int attn_query_tile(int heads, int kv_heads);     // tokens per query tile of the multi-token kernel

// ---- recurrent.cu ----------------------------------------------------------------------------------
enum RecKind : int { REC_GLA = 0, REC_DELTA = 1, REC_HGRN2 = 2, REC_WKV = 3, REC_GENERAL = 4 };
struct RecArgs {
    int kind;
    const void *proj;   // [rows, ldp]
    int ldp, q_off, k_off, v_off, b_off, g_off;  // b: step-size column (delta), removal rates (general); g: output gate inside proj (all but delta)
    const void *z;      // [rows, ldz]: decay logits at z_off, output gate at zg_off (delta); HGRN2: proj itself
    int ldz, z_off, zg_off;
    int heads, kv_heads, DK, DV;  // padded head sizes
    int dim, vdim;      // true head sizes
    float tau, out_scale, eps;
    const float *conv_q, *conv_k, *conv_v;  // [channels][taps] (padded channels), taps = 0: no convolution
    int taps;
    const float *decay_bias;  // [heads * DK]
    const float *a_log;       // [heads] (delta)
    const float *norm_w;      // [DV], or [heads * DV]: norm_stride is DV then
    int norm_stride;
    const float *removal_bias;  // [heads * DK], and the rate of the decay (general)
    float rate;
    const float *bonus;       // [heads * DK] weight of the current token (WKV)
    const float *lower;       // [heads * DK] lower bound of the forget gate (HGRN2)
    int shift_width;          // width of the previous token's input kept in the state (WKV)
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

// ---- attn_latent.cu ----------------------------------------------------------------------------------
// Latent attention.  A page row is [latent c, padded to KR | rotated key part, padded to RR | 8 unused], LDR elements.
// On the latents ("absorbed"): scores q~ . c + q_rot . k_rot with q~ = W_uk^T q per head, the output a weighted sum of c.
// Written out: keys [W_uk c | k_rot] and values W_uv c per head in a workspace, for entries with many query rows.
struct LatentEntry {
    int entry, key0, n_keys, row0;  // the keys of positions [key0, key0 + n_keys) in workspace rows [row0, ..)
};
struct LatentArgs {
    const void *proj;   // [rows, ldp]: query latent at dq_off, key latent at c_off, rotated part behind it at r_off
    int ldp, dq_off, c_off, r_off;
    int q_rank, kv_rank, rot_dim, half;
    float eps, scale;
    const float *dq_norm, *dkv_norm;
    void *cq;           // [rows, ldcq]
    int ldcq, own_cache;
    int KR, RR, LDR;
    void *kv;           // pages [block][16][LDR]
    const int *table;
    int n_blocks, mbs;
    const float2 *cs;   // [rows][half]
    const void *q;      // [rows, ldq], head h at h * DQ: [dim, padded to DP | rot_dim ...]
    int ldq, DQ, DP, dim;
    void *qa;           // [rows, heads * KR]: q~, replaced by the weighted sums
    int heads, window;
    // written-out form
    void *cx;           // [workspace rows][KR + RR]
    const void *kvx;    // [workspace rows][ldx]: keys at h * DP, values at heads * DP + h * DVm
    int ldx, DVm, vdim;
    void *out;          // [rows, ldo], head h at out_off + h * DVm
    int ldo, out_off;
    int sm_count;
    int *status;
};
int latent_padded_rank(int kv_rank);   // KR; 0: not supported by the tensor-core kernel
int latent_padded_rot(int rot_dim);
bool latent_expandable(int dim, int rot_dim, int vdim);
int32_t launch_latent_prep(bool f32, const StepDesc &d, const LatentArgs &a, int pdl, cudaStream_t st);
int32_t launch_latent_attention(bool f32, const StepDesc &d, const LatentArgs &a, int pdl, cudaStream_t st);
int32_t launch_latent_gather(const StepDesc &d, const LatentArgs &a, int first, int n, int max_keys, int pdl, cudaStream_t st);
int32_t launch_latent_tiles(const StepDesc &d, const LatentArgs &a, int first_tile, int n_tiles, int pdl, cudaStream_t st);
constexpr int kLatentTile = 64;  // query tokens per tile of the written-out form

}  // namespace mix
}  // namespace jgpt
