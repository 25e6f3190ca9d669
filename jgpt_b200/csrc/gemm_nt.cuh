// Projections with weights in [out, in] layout: C[M, N] = A[M, K] . W[N, K]^T, bf16 operands with fp32 accumulation or
// plain fp32.  Host-side interface of gemm_nt.cu (small M, and fp32) and gemm_nt_umma.cu (large M, tcgen05).
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace jgpt {
namespace nt {

// What happens to a finished sum.
enum Epilogue : int {
    EPI_STORE = 0,     // C (activation type) = sum
    EPI_ADD_F32 = 1,   // C (fp32) = residual + column factor * sum; every element is read and written by one thread
    EPI_SCALE_F32 = 2, // C (fp32) = sum * scale
    EPI_GATE_GELU = 3, // W rows alternate in groups of 16: 16 of the gate, 16 of the linear part; C [M, N / 2] = gelu(gate) * linear
    EPI_ACT = 4,       // C (activation type) = act(sum), the function picked per product
};
enum Activation : int { ACT_NONE = 0, ACT_TANH = 1, ACT_XIELU = 2 };

struct Problem {
    const void *A;     // [M, lda]
    const void *W;     // [N, ldw]
    void *C;           // [M, ldc]
    const int *rowsel; // optional: row m of A is rowsel[m] (not for the large-M kernel)
    int M, N, K, lda, ldw, ldc;
    float scale = 1.f;
    // Segments: columns [s seg_n, (s + 1) seg_n) read the operand at A + s a_seg (elements) and land at column n + s c_seg of C.
    // a_seg is a multiple of lda (other rows) or less than lda (other columns of the same rows).  0: one segment.
    int seg_n = 0, c_seg = 0;
    long long a_seg = 0;
    const float *res = nullptr, *colscale = nullptr;  // EPI_ADD_F32: residual [M, ldc] (null: C itself), factor per column (null: 1)
    int act = ACT_NONE;                               // EPI_ACT
    float p0 = 0.f, p1 = 0.f;                         // its parameters
    int segments() const { return seg_n > 0 ? (N + seg_n - 1) / seg_n : 1; }
    int segment_cols() const { return seg_n > 0 ? seg_n : N; }
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
__device__ __forceinline__ float activate(int act, float p0, float p1, float z) {
    return act == ACT_XIELU ? xielu(z, p0, p1) : (act == ACT_TANH ? tanhf(z) : z);
}
__device__ __forceinline__ float activate_fast(int act, float p0, float p1, float z) {
    return act == ACT_XIELU ? xielu_fast(z, p0, p1) : (act == ACT_TANH ? tanhf(z) : z);
}

// Runs 1 or 2 independent products (same M) in one launch.  K, lda, ldw and (bf16) the operand addresses must allow
// 16-byte row chunks: multiples of 8 elements (bf16) or 4 (fp32).  pdl: bit 0 = this launch may start early and waits
// itself; bit 1 = it lets the next launch in.
int32_t launch_bf16(const Ctx *ctx, const Problem *p, int n, Epilogue epi, int pdl, cudaStream_t st);
int32_t launch_f32(const Problem *p, int n, Epilogue epi, cudaStream_t st);

// From this many rows on launch_bf16 takes the tcgen05 kernel.
int umma_min_rows();
int32_t launch_bf16_umma(const Ctx *ctx, const Problem &p, Epilogue epi, int pdl, cudaStream_t st);

}  // namespace nt
}  // namespace jgpt
