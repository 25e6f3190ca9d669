// Paged attention of the layered decoder: query heads in groups that share a key head, head sizes up to 256 (padded to a
// multiple of 32), a visibility rule by chunks of positions, an optional output gate per head.
//
//   attn_append_kernel   rows of K and V into the pages (in the cache's type; no rotation)
//   attn_rows_kernel     one warp per (row, head), any type: the exact fp32 mode
#include "mixers.cuh"

#include <algorithm>

#include "ptx.cuh"

namespace jgpt {
namespace mix {

__device__ __forceinline__ float act_load(const __nv_bfloat16 *p) { return __bfloat162float(*p); }
__device__ __forceinline__ float act_load(const float *p) { return *p; }
__device__ __forceinline__ void act_store(__nv_bfloat16 *p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void act_store(float *p, float v) { *p = v; }

// Physical block of a position, or -1 (recorded in the status word).
__device__ __forceinline__ int page_of(const AttnArgs &a, int seq, int pos) {
    const int b = pos / kBlockTokens;
    if (b < 0 || b >= a.mbs) {
        atomicOr(a.status, DEV_STATUS_BAD_POSITION);
        return -1;
    }
    const int phys = a.table[(size_t)seq * a.mbs + b];
    if (phys < 0 || phys >= a.n_blocks) {
        atomicOr(a.status, DEV_STATUS_BAD_BLOCK);
        return -1;
    }
    return phys;
}
__host__ __device__ __forceinline__ int first_visible(int pos, int chunk) { return chunk > 0 ? pos / chunk * chunk : 0; }

// One thread moves 16 bytes of one (row, key head) of K and of V.
template <class AT>
__global__ void __launch_bounds__(256) attn_append_kernel(const AttnArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int rows,
                                                          int pdl) {
    constexpr int E = 16 / sizeof(AT);
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    const int cpr = a.D / E;
    const long long gid = (long long)blockIdx.x * 256 + threadIdx.x;
    if (gid >= (long long)rows * a.kv_heads * cpr) return;
    const int c = (int)(gid % cpr), g = (int)(gid / cpr % a.kv_heads), r = (int)(gid / ((long long)cpr * a.kv_heads));
    const int p = pos[r], phys = page_of(a, seq[r], p);
    if (phys < 0) return;
    const AT *src = reinterpret_cast<const AT *>(a.proj) + (size_t)r * a.ldp + g * a.D + c * E;
    AT *dst = reinterpret_cast<AT *>(a.kv) + ((size_t)phys * a.kv_heads + g) * (2 * kBlockTokens * a.D) + (size_t)(p % kBlockTokens) * a.D + c * E;
    *reinterpret_cast<uint4 *>(dst) = *reinterpret_cast<const uint4 *>(src + a.k_off);
    *reinterpret_cast<uint4 *>(dst + kBlockTokens * a.D) = *reinterpret_cast<const uint4 *>(src + a.v_off);
}

// One warp per (row, query head): lane l holds elements l, l + 32, ... of q and of the output.
template <class AT>
__global__ void __launch_bounds__(256) attn_rows_kernel(const AttnArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int rows) {
    constexpr int MAXE = 8;
    const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= rows * a.heads) return;
    const int r = item / a.heads, h = item % a.heads, g = h / (a.heads / a.kv_heads), ne = a.D / 32;
    const AT *proj = reinterpret_cast<const AT *>(a.proj) + (size_t)r * a.ldp;
    float q[MAXE], o[MAXE];
#pragma unroll
    for (int e = 0; e < MAXE; e++) q[e] = e < ne ? act_load(proj + a.q_off + h * a.D + lane + 32 * e) * a.scale : 0.f, o[e] = 0.f;
    float m = -INFINITY, l = 0.f;
    const int p = pos[r], s = seq[r];
    for (int j = first_visible(p, a.chunk); j <= p; j++) {
        const int phys = page_of(a, s, j);
        if (phys < 0) break;
        const AT *k = reinterpret_cast<const AT *>(a.kv) + ((size_t)phys * a.kv_heads + g) * (2 * kBlockTokens * a.D) +
                      (size_t)(j % kBlockTokens) * a.D + lane;
        float d = 0.f;
#pragma unroll
        for (int e = 0; e < MAXE; e++)
            if (e < ne) d = fmaf(q[e], act_load(k + 32 * e), d);
#pragma unroll
        for (int off = 16; off >= 1; off >>= 1) d += __shfl_xor_sync(0xffffffffu, d, off);
        const float mn = fmaxf(m, d), f = expf(m - mn), w = expf(d - mn);
        m = mn, l = l * f + w;
#pragma unroll
        for (int e = 0; e < MAXE; e++)
            if (e < ne) o[e] = fmaf(w, act_load(k + kBlockTokens * a.D + 32 * e), o[e] * f);
    }
    float f = (l > 0.f ? 1.f / l : 0.f) * a.out_scale;
    if (a.g_off >= 0) f *= 1.f / (1.f + expf(-act_load(proj + a.g_off + h)));
    AT *out = reinterpret_cast<AT *>(a.out) + (size_t)r * a.ldo + a.out_off + h * a.D + lane;
#pragma unroll
    for (int e = 0; e < MAXE; e++)
        if (e < ne) act_store(out + 32 * e, o[e] * f);
}

int attn_padded_head(int dim, int vdim) {
    const int d = std::max(dim, vdim);
    for (int p : {32, 64, 96, 128, 192, 256})
        if (d <= p) return dim > 0 && vdim > 0 ? p : 0;
    return 0;
}
int attn_query_tile(int heads, int kv_heads) { return std::max(1, 64 / (heads / kv_heads)); }
uint64_t attn_partial_floats(int rows, int heads, int D) { return 0; }

template <class AT>
static int32_t rows_attention(const StepDesc &d, const AttnArgs &a, int pdl, cudaStream_t st) {
    const long long total = (long long)d.rows * a.kv_heads * (a.D / (16 / (int)sizeof(AT)));
    attn_append_kernel<AT><<<(unsigned)((total + 255) / 256), 256, 0, st>>>(a, d.seq, d.pos, d.rows, 0);
    attn_rows_kernel<AT><<<(unsigned)((d.rows * (long long)a.heads + 7) / 8), 256, 0, st>>>(a, d.seq, d.pos, d.rows);
    JGPT_CUDA_TRY(cudaGetLastError());
    return JGPT_OK;
}

int32_t launch_attention(bool f32, const StepDesc &d, const AttnArgs &a, int pdl, cudaStream_t st) {
    return f32 ? rows_attention<float>(d, a, pdl, st) : rows_attention<__nv_bfloat16>(d, a, pdl, st);
}

}  // namespace mix
}  // namespace jgpt
