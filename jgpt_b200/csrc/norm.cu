// Embedding and layer norm of the layered decoder.  The residual stream and the norms are fp32.
#include "mixers.cuh"
#include "ptx.cuh"

namespace jgpt {
namespace mix {

constexpr int kNormThreads = 256;

__device__ __forceinline__ void store_act(__nv_bfloat16 *p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void store_act(float *p, float v) { *p = v; }
__device__ __forceinline__ float load_act(const __nv_bfloat16 *p) { return __bfloat162float(*p); }
__device__ __forceinline__ float load_act(const float *p) { return *p; }

__device__ __forceinline__ float block_sum(float v, float *red) {
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
    __syncthreads();  // the previous use of red is over
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < kNormThreads / 32; w++) s += red[w];
    return s;
}

// (mean, 1 / sqrt(variance + eps)) of the row in shared memory; the variance from the squared deviations.
__device__ __forceinline__ float2 row_stats(const float *row, int W, float eps, float *red) {
    float s = 0.f;
    for (int j = threadIdx.x; j < W; j += kNormThreads) s += row[j];
    const float mean = block_sum(s, red) / (float)W;
    float q = 0.f;
    for (int j = threadIdx.x; j < W; j += kNormThreads) {
        const float d = row[j] - mean;
        q += d * d;
    }
    return make_float2(mean, 1.f / sqrtf(block_sum(q, red) / (float)W + eps));
}

template <class AT>
__global__ void __launch_bounds__(kNormThreads) embed_norm_kernel(const int *__restrict__ tok, const int *__restrict__ pos,
                                                                  const AT *__restrict__ embed, int ld_embed,
                                                                  const AT *__restrict__ pos_table, int ld_pos, float scale,
                                                                  const NormW en, const NormW nn, float eps, float *__restrict__ x,
                                                                  AT *__restrict__ h, int W, int ldh, int vocab, int max_pos, int *status,
                                                                  int pdl) {
    extern __shared__ float row[];
    __shared__ float red[kNormThreads / 32];
    const int r = blockIdx.x;
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    int t = tok[r], p = pos[r];
    if (t < 0 || t >= vocab || p < 0 || (pos_table && p >= max_pos)) {
        if (threadIdx.x == 0) atomicOr(status, DEV_STATUS_BAD_POSITION);
        t = p = 0;
    }
    for (int j = threadIdx.x; j < W; j += kNormThreads) {
        float v = load_act(embed + (size_t)t * ld_embed + j) * scale;
        if (pos_table) v += load_act(pos_table + (size_t)p * ld_pos + j);
        row[j] = v;
    }
    __syncthreads();
    if (en.gamma) {
        const float2 s = row_stats(row, W, eps, red);
        for (int j = threadIdx.x; j < W; j += kNormThreads) row[j] = (row[j] - s.x) * s.y * en.gamma[j] + en.beta[j];
        __syncthreads();
    }
    const float2 s = row_stats(row, W, eps, red);
    for (int j = threadIdx.x; j < ldh; j += kNormThreads) {
        if (j < W) x[(size_t)r * W + j] = row[j];
        store_act(h + (size_t)r * ldh + j, j < W ? (row[j] - s.x) * s.y * nn.gamma[j] + nn.beta[j] : 0.f);
    }
}

template <class AT>
__global__ void __launch_bounds__(kNormThreads) layer_norm_kernel(const float *__restrict__ x, const int *__restrict__ rowsel, const NormW w,
                                                                  float eps, AT *__restrict__ h, int W, int ldh, int pdl) {
    extern __shared__ float row[];
    __shared__ float red[kNormThreads / 32];
    const int r = blockIdx.x;
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    const float *xr = x + (size_t)(rowsel ? rowsel[r] : r) * W;
    if ((W & 3) == 0) {
        for (int j = threadIdx.x; j < W / 4; j += kNormThreads)
            reinterpret_cast<float4 *>(row)[j] = reinterpret_cast<const float4 *>(xr)[j];
    } else {
        for (int j = threadIdx.x; j < W; j += kNormThreads) row[j] = xr[j];
    }
    __syncthreads();
    const float2 s = row_stats(row, W, eps, red);
    for (int j = threadIdx.x; j < ldh; j += kNormThreads)
        store_act(h + (size_t)r * ldh + j, j < W ? (row[j] - s.x) * s.y * w.gamma[j] + w.beta[j] : 0.f);
}

template <class... Args>
static int32_t launch(void (*kern)(Args...), int grid, size_t smem, int pdl, cudaStream_t st, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = dim3((unsigned)grid), cfg.blockDim = dim3(kNormThreads), cfg.dynamicSmemBytes = smem, cfg.stream = st;
    cfg.attrs = attr, cfg.numAttrs = (pdl & 1) ? 1 : 0;
    JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, kern, args...));
    return JGPT_OK;
}

int32_t launch_embed(bool f32, const StepDesc &d, const void *embed, int ld_embed, const void *pos_table, int ld_pos, float scale,
                     NormW en, NormW nn, float eps, float *x, void *h, int W, int ldh, int vocab, int max_pos, int *status, int pdl,
                     cudaStream_t st) {
    const size_t smem = sizeof(float) * (size_t)W;
    JGPT_REQUIRE(smem <= 48 * 1024 - 256, JGPT_ERR_UNSUPPORTED, "width %d", W);
    if (f32)
        return launch(embed_norm_kernel<float>, d.rows, smem, pdl, st, d.tok, d.pos, (const float *)embed, ld_embed, (const float *)pos_table,
                      ld_pos, scale, (const NormW)en, (const NormW)nn, eps, x, (float *)h, W, ldh, vocab, max_pos, status, pdl);
    return launch(embed_norm_kernel<__nv_bfloat16>, d.rows, smem, pdl, st, d.tok, d.pos, (const __nv_bfloat16 *)embed, ld_embed,
                  (const __nv_bfloat16 *)pos_table, ld_pos, scale, (const NormW)en, (const NormW)nn, eps, x, (__nv_bfloat16 *)h, W, ldh, vocab,
                  max_pos, status, pdl);
}

int32_t launch_layer_norm(bool f32, const float *x, const int *rowsel, NormW w, float eps, void *h, int rows, int W, int ldh, int pdl,
                          cudaStream_t st) {
    const size_t smem = sizeof(float) * (size_t)W;
    JGPT_REQUIRE(smem <= 48 * 1024 - 256, JGPT_ERR_UNSUPPORTED, "width %d", W);
    if (f32) return launch(layer_norm_kernel<float>, rows, smem, pdl, st, x, rowsel, (const NormW)w, eps, (float *)h, W, ldh, pdl);
    return launch(layer_norm_kernel<__nv_bfloat16>, rows, smem, pdl, st, x, rowsel, (const NormW)w, eps, (__nv_bfloat16 *)h, W, ldh, pdl);
}

}  // namespace mix
}  // namespace jgpt
