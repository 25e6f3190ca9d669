// Projections with weights in [out, in] layout: C[M, N] = A[M, K] . W[N, K]^T, bf16 operands with fp32 accumulation or
// plain fp32.  Host-side interface of gemm_nt.cu (small M, and fp32) and gemm_nt_umma.cu (large M, tcgen05).
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace jgpt {
namespace nt {

// What happens to a finished sum.
enum Epilogue : int {
    EPI_STORE = 0,     // C (activation type) = sum + bias
    EPI_ADD_F32 = 1,   // C (fp32) = residual factor * residual + column factor * sum; every element is read and written by one thread
    EPI_SCALE_F32 = 2, // C (fp32) = sum * scale
    EPI_GATE = 3,      // W rows alternate in groups of 16: 16 of the gate, 16 of the linear part; C [M, N / 2] = act(gate) * linear
    EPI_ACT = 4,       // C (activation type) = act(sum), the function picked per product
    EPI_ACT_SOME = 5,  // the same for columns [act_from, act_to); the others get the bias (which is set) alone
};
enum Activation : int { ACT_NONE = 0, ACT_TANH = 1, ACT_XIELU = 2, ACT_GELU = 3, ACT_RELU = 4, ACT_RELU2 = 5 };

// Rows in groups with weights of their own (experts).  The rows of C lie group by group; a tile covers rows [row0, row_end) of
// one group, at most `rows` of them, and the weights of a group start w_group elements behind those of the group before.  Row m of
// the operand is rowsel[src0 + m - row0], or m without rowsel.  Tiles and their number are written by the device.
struct RowTile {
    int group, row0, row_end, src0;
};
struct RowGroups {
    const RowTile *tiles = nullptr;
    const int *n_tiles = nullptr;
    int max_tiles = 0, rows = 0, n_groups = 0;
    int a_rows = 0;      // rows of A
    long long w_group = 0;
    bool early = false;  // the tiles are older than the launch in front of this one
};

struct Problem {
    const void *A;     // [M, lda]
    const void *W;     // [N, ldw]
    void *C;           // [M, ldc]
    const int *rowsel; // optional: row m of A is rowsel[m] (not for the large-M kernel)
    int M, N, K, lda, ldw, ldc;
    float scale = 1.f;
    // Segments: columns [s seg_n, (s + 1) seg_n) read the operand at A + s a_seg (elements) and land at column n + s c_seg of C.
    // a_seg is a multiple of lda (other rows) or less than lda (other columns of the same rows).  0: one segment.
    // From segment a_cap on the operand stays where it is.
    int seg_n = 0, c_seg = 0, a_cap = 1 << 30;
    long long a_seg = 0;
    const float *res = nullptr, *colscale = nullptr;  // EPI_ADD_F32: residual [M, ldc] (null: C itself), factor per column (null: 1)
    int act = ACT_NONE;                               // EPI_ACT
    float p0 = 0.f, p1 = 0.f;                         // its parameters
    int act_from = 0, act_to = 0;                     // EPI_ACT_SOME
    const float *bias = nullptr;                      // EPI_STORE, EPI_ACT_SOME: per column
    float res_scale = 1.f;                            // EPI_ADD_F32
    RowGroups grp;                                    // tiles set: rows in groups (EPI_STORE, EPI_ACT; one segment)
    int segments() const { return seg_n > 0 ? (N + seg_n - 1) / seg_n : 1; }
    int segment_cols() const { return seg_n > 0 ? seg_n : N; }
    int column_tiles(int bn) const {  // the last segment may be shorter
        const int s = segments(), c = segment_cols();
        return (s - 1) * ((c + bn - 1) / bn) + (N - (s - 1) * c + bn - 1) / bn;
    }
};

// gelu(z) in its tanh form, 0.5 z (1 + tanh(u)) = z / (1 + exp(-2 u)), u = sqrt(2 / pi) (z + 0.044715 z^3).
__device__ __forceinline__ float gelu_tanh(float z) {
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return z / (1.f + expf(-2.f * u));
}

// xIELU: a z^2 + z / 2 for positive z, b (e^z - 1 - z) + z / 2 otherwise.
__device__ __forceinline__ float xielu(float z, float a, float b) { return 0.5f * z + (z > 0.f ? a * z * z : b * (expm1f(z) - z)); }
// The same with the fast exponential, for results that are rounded to bf16: e^z - 1 - z from its series near 0.
__device__ __forceinline__ float xielu_fast(float z, float a, float b) {
    const float e = z > -0.03125f ? z * z * fmaf(z, fmaf(z, 1.f / 24.f, 1.f / 6.f), 0.5f) : __expf(z) - 1.f - z;
    return fmaf(0.5f, z, z > 0.f ? a * z * z : b * e);
}
// FAST: for results that are rounded to bf16.
template <bool FAST>
__device__ __forceinline__ float activate(int act, float p0, float p1, float z) {
    switch (act) {
        case ACT_XIELU: return FAST ? xielu_fast(z, p0, p1) : xielu(z, p0, p1);
        case ACT_TANH: return tanhf(z);
        case ACT_GELU: return gelu_tanh(z);
        case ACT_RELU: return fmaxf(z, 0.f);
        case ACT_RELU2: z = fmaxf(z, 0.f); return z * z;
        default: return z;
    }
}

// Runs 1 or 2 independent products (same M) in one launch.  K, lda, ldw and (bf16) the operand addresses must allow
// 16-byte row chunks: multiples of 8 elements (bf16) or 4 (fp32).  pdl: bit 0 = this launch may start early and waits
// itself; bit 1 = it lets the next launch in.  Of two products the first may have rows in groups; M is then the number of rows
// the other one has.
int32_t launch_bf16(const Ctx *ctx, const Problem *p, int n, Epilogue epi, int pdl, cudaStream_t st);
int32_t launch_f32(const Problem *p, int n, Epilogue epi, cudaStream_t st);

// From this many rows on launch_bf16 takes the tcgen05 kernel.
int umma_min_rows();
// Rows of a tile (RowGroups::rows) for products of `rows` rows, each of which is in `copies` of the groups; kLargeTile: the large-M
// kernel, whose operand holds the rows group by group.
constexpr int kLargeTile = 128;
int group_tile_rows(bool f32, int rows, int copies, int groups);
int32_t launch_bf16_umma(const Ctx *ctx, const Problem &p, Epilogue epi, int pdl, cudaStream_t st);

}  // namespace nt
}  // namespace jgpt
