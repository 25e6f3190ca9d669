// Embedding and norms of the layered decoder: layer norm over a plain residual, RMS norm over a residual that may be the
// embedding, a weighted sum of the earlier layers' results, and mixed with the previous token's row.  The residual stream and
// the norms are fp32.
#include <algorithm>
#include <type_traits>

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
__global__ void __launch_bounds__(kNormThreads) layer_norm_kernel(const float *x, const int *__restrict__ rowsel, const NormW w,
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

// ------------------------------------------------------------------------------------------------
// RMS norm
// ------------------------------------------------------------------------------------------------
// Row `src` of the residual into shared memory (and to x), its 1 / rms returned.
template <class AT, bool EMBED>
__device__ __forceinline__ float residual_row(const RowSource &s, const int *__restrict__ tok, int src, float eps, float *row, float *x, int W, float *red, int *status) {
    float q = 0.f;
    if (EMBED) {
        int t = tok[src];
        if (t < 0 || t >= s.vocab) {
            if (threadIdx.x == 0) atomicOr(status, DEV_STATUS_BAD_POSITION);
            t = 0;
        }
        const AT *e = reinterpret_cast<const AT *>(s.embed) + (size_t)t * s.ld_embed;
        for (int j = threadIdx.x; j < W; j += kNormThreads) {
            const float v = load_act(e + j) * s.embed_scale;
            row[j] = v, q += v * v;
            if (x) x[(size_t)src * W + j] = v;
        }
    } else if ((W & 3) == 0) {
        const float *base = s.slots + (size_t)src * W;
        for (int j = threadIdx.x * 4; j < W; j += kNormThreads * 4) {
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (!s.weights) v = *reinterpret_cast<const float4 *>(base + j);
            else {
#pragma unroll 8
                for (int i = 0; i < s.n_slots; i++) {
                    const float4 y = *reinterpret_cast<const float4 *>(base + i * s.slot_stride + j);
                    const float w = __ldg(s.weights + i);
                    v.x = fmaf(w, y.x, v.x), v.y = fmaf(w, y.y, v.y), v.z = fmaf(w, y.z, v.z), v.w = fmaf(w, y.w, v.w);
                }
            }
            *reinterpret_cast<float4 *>(row + j) = v;
            if (x) *reinterpret_cast<float4 *>(x + (size_t)src * W + j) = v;
            q += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        const float *base = s.slots + (size_t)src * W;
        for (int j = threadIdx.x; j < W; j += kNormThreads) {
            float v = s.weights ? 0.f : base[j];
            if (s.weights)
                for (int i = 0; i < s.n_slots; i++) v = fmaf(__ldg(s.weights + i), base[i * s.slot_stride + j], v);
            row[j] = v, q += v * v;
            if (x) x[(size_t)src * W + j] = v;
        }
    }
    return 1.f / sqrtf(block_sum(q, red) / (float)W + eps);
}

template <class AT, bool EMBED>
__global__ void __launch_bounds__(kNormThreads) residual_norm_kernel(const StepDesc d, const RowSource s, const int *__restrict__ rowsel,
                                                                     const float *__restrict__ gamma, float eps, float *x, AT *__restrict__ h,
                                                                     const ShiftArgs sh, int W, int ldh, int *status, int pdl) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[kNormThreads / 32];
    const int r = blockIdx.x;
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    const int src = rowsel ? rowsel[r] : r;
    const float inv = residual_row<AT, EMBED>(s, d.tok, src, eps, row, x, W, red, status);
    if (EMBED) {
        for (int k = 0; k < s.n_rot; k++)
            for (int i = threadIdx.x; i < s.rot[k].half; i += kNormThreads) {
                double sn, cs;
                sincos((double)d.pos[src] * s.rot[k].freq[i], &sn, &cs);
                s.rot[k].out[(size_t)src * s.rot[k].half + i] = make_float2((float)cs * s.rot[k].mag, (float)sn * s.rot[k].mag);
            }
    }
    if (!h) return;
    if (!sh.mu[0]) {
        for (int j = threadIdx.x; j < ldh; j += kNormThreads) store_act(h + (size_t)r * ldh + j, j < W ? (gamma ? row[j] * inv * gamma[j] : row[j]) : 0.f);
        return;
    }
    // the row before: recomputed the same way inside an entry, read from the state in front of it
    float *before = row + (W + 3) / 4 * 4;
    const Seg sg = d.segs[d.ent[src]];
    if (sg.seq < 0 || sg.seq >= sh.max_seqs) {
        if (threadIdx.x == 0) atomicOr(status, DEV_STATUS_BAD_SEQ);
        return;
    }
    float *hist = reinterpret_cast<float *>(sh.state + (uint64_t)sg.seq * sh.state_stride);
    const bool first = src == sg.row0, last = src == sg.row0 + sg.T - 1;
    float binv = 0.f;
    if (!first) binv = residual_row<AT, EMBED>(s, d.tok, src - 1, eps, before, nullptr, W, red, status);
    for (int j = threadIdx.x; j < ldh; j += kNormThreads) {
        float v = 0.f, dv = 0.f;
        if (j < W) {
            v = row[j] * inv * gamma[j];
            const float p = first ? (sg.pos0 > 0 ? hist[(size_t)sg.conv_set * W + j] : 0.f) : before[j] * binv * gamma[j];
            dv = p - v;
            if (last) hist[(size_t)(1 - sg.conv_set) * W + j] = v;
        }
#pragma unroll
        for (int m = 0; m < 5; m++) store_act(h + m * sh.out_stride + (size_t)r * ldh + j, j < W ? fmaf(dv, sh.mu[m][j], v) : 0.f);
    }
}

int32_t launch_residual_norm(bool f32, const StepDesc &d, const RowSource &s, const int *rowsel, int rows, const float *gamma, float eps, float *x,
                             void *h, const ShiftArgs &sh, int W, int ldh, int *status, int pdl, cudaStream_t st) {
    const size_t smem = sizeof(float) * (size_t)((W + 3) / 4 * 4) * (sh.mu[0] ? 2 : 1);
    JGPT_REQUIRE(smem <= 48 * 1024 - 256, JGPT_ERR_UNSUPPORTED, "width %d", W);
    auto run = [&](auto kern, auto *act) {
        return launch(kern, rows, smem, pdl, st, (const StepDesc)d, (const RowSource)s, rowsel, gamma, eps, x, (decltype(act))h, (const ShiftArgs)sh, W, ldh,
                      status, pdl);
    };
    if (f32) return s.embed ? run(residual_norm_kernel<float, true>, (float *)nullptr) : run(residual_norm_kernel<float, false>, (float *)nullptr);
    return s.embed ? run(residual_norm_kernel<__nv_bfloat16, true>, (__nv_bfloat16 *)nullptr)
                   : run(residual_norm_kernel<__nv_bfloat16, false>, (__nv_bfloat16 *)nullptr);
}

// ------------------------------------------------------------------------------------------------
// RMS norm behind a sum
// ------------------------------------------------------------------------------------------------
__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16 *p) {
    const uint2 u = *reinterpret_cast<const uint2 *>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16 *p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
}
__device__ __forceinline__ void add_scaled(float4 &s, float w, const float4 &v) {
    s.x = fmaf(w, v.x, s.x), s.y = fmaf(w, v.y, s.y), s.z = fmaf(w, v.z, s.z), s.w = fmaf(w, v.w, s.w);
}

constexpr int kMaxTop = 32;

template <class AT, bool MOE>
__global__ void __launch_bounds__(kNormThreads) post_norm_kernel(float *x, const float *__restrict__ gamma, float eps, AT *__restrict__ h, const MoeSum m,
                                                                 int W, int ldh, int pdl) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[kNormThreads / 32], weight[kMaxTop];
    __shared__ long long from[kMaxTop];
    const int r = blockIdx.x, tid = threadIdx.x;
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    float *xr = x + (size_t)r * W;
    const AT *out = reinterpret_cast<const AT *>(m.out), *shared = reinterpret_cast<const AT *>(m.shared) + (size_t)r * m.ld;
    float keep = 1.f, gate = 0.f;
    if (MOE) {
        if (tid < m.top) {
            const RouteSlot s = m.slots[(size_t)r * m.top + tid];
            const bool ok = s.expert >= 0 && s.rank >= 0 && s.rank < m.cap;
            weight[tid] = ok ? s.weight : 0.f, from[tid] = ok ? (long long)(m.offsets[s.expert] + s.rank) * m.ld : -1;
        }
        const float2 w = m.row_weights[r];
        keep = m.alpha + w.x, gate = w.y;
        __syncthreads();
    }
    float q = 0.f;
    if ((W & 3) == 0) {
        for (int j = tid * 4; j < W; j += kNormThreads * 4) {
            float4 v = load4(xr + j);
            if (MOE) {
                v.x *= keep, v.y *= keep, v.z *= keep, v.w *= keep;
#pragma unroll 8
                for (int s = 0; s < m.top; s++)
                    if (from[s] >= 0) add_scaled(v, weight[s], load4(out + from[s] + j));
                if (m.shared) add_scaled(v, gate, load4(shared + j));
            }
            store4(row + j, v);
            q += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int j = tid; j < W; j += kNormThreads) {
            float v = xr[j];
            if (MOE) {
                v *= keep;
                for (int s = 0; s < m.top; s++)
                    if (from[s] >= 0) v = fmaf(weight[s], load_act(out + from[s] + j), v);
                if (m.shared) v = fmaf(gate, load_act(shared + j), v);
            }
            row[j] = v, q += v * v;
        }
    }
    const float inv = 1.f / sqrtf(block_sum(q, red) / (float)W + eps);
    AT *hr = h + (size_t)r * ldh;
    if ((W & 3) == 0) {
        for (int j = tid * 4; j < W; j += kNormThreads * 4) {
            const float4 v = load4(row + j), g = load4(gamma + j), y = make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w);
            store4(xr + j, y), store4(hr + j, y);
        }
        for (int j = W + tid; j < ldh; j += kNormThreads) store_act(hr + j, 0.f);
        return;
    }
    for (int j = tid; j < ldh; j += kNormThreads) {
        const float y = j < W ? row[j] * inv * gamma[j] : 0.f;
        if (j < W) xr[j] = y;
        store_act(hr + j, y);
    }
}

int32_t launch_post_norm(bool f32, float *x, int rows, const float *gamma, float eps, void *h, const MoeSum &m, int W, int ldh, int pdl, cudaStream_t st) {
    const size_t smem = sizeof(float) * (size_t)((W + 3) / 4 * 4);
    JGPT_REQUIRE(smem <= 47 * 1024 && m.top <= kMaxTop, JGPT_ERR_UNSUPPORTED, "width %d, %d experts per token", W, m.top);
    auto run = [&](auto kern, auto *act) { return launch(kern, rows, smem, pdl, st, x, gamma, eps, (decltype(act))h, (const MoeSum)m, W, ldh, pdl); };
    if (f32) return m.out ? run(post_norm_kernel<float, true>, (float *)nullptr) : run(post_norm_kernel<float, false>, (float *)nullptr);
    return m.out ? run(post_norm_kernel<__nv_bfloat16, true>, (__nv_bfloat16 *)nullptr) : run(post_norm_kernel<__nv_bfloat16, false>, (__nv_bfloat16 *)nullptr);
}

// ------------------------------------------------------------------------------------------------
// RMS norms on both sides of a part
// ------------------------------------------------------------------------------------------------
__device__ __forceinline__ float dot4(const float4 &v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
template <class AT>
__device__ __forceinline__ float sigmoid_act(float z) {
    return sizeof(AT) == 4 ? 1.f / (1.f + expf(-z)) : __fdividef(1.f, 1.f + __expf(-z));
}

// A block takes `per` rows one after the other, 4 NV columns per thread in registers: the row in front of each is at hand for the
// token shift.  Only the row in front of the block's first one is computed twice, so x is read and written in different arrays.
template <class AT, bool EMBED, int NV>
__global__ void __launch_bounds__(kNormThreads) part_norm_kernel(const StepDesc d, const RowSource s, const PartNorm a, const int *rowsel, int rows, int per,
                                                                 float eps, int W, int ldw, int *status, int pdl) {
    __shared__ float red[kNormThreads / 32];
    const int tid = threadIdx.x, r0 = blockIdx.x * per, r1 = min(rows, r0 + per);
    if (pdl & 2) griddep_launch_dependents();
    int first = r0;
    if (a.shifted && r0 > d.segs[d.ent[r0]].row0) first = r0 - 1;
    if (pdl & 1) griddep_wait();
    float4 before[NV];
    for (int r = first; r < r1; r++) {
        const int src = rowsel ? rowsel[r] : r;
        const bool own = r >= r0;
        float4 x[NV];
        if (EMBED) {
            int t = d.tok[src];
            if (t < 0 || t >= s.vocab) {
                if (tid == 0) atomicOr(status, DEV_STATUS_BAD_POSITION);
                t = 0;
            }
            const AT *e = reinterpret_cast<const AT *>(s.embed) + (size_t)t * s.ld_embed;
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int j = (tid + i * kNormThreads) * 4;
                x[i] = j < ldw ? load4(e + j) : make_float4(0.f, 0.f, 0.f, 0.f);
                x[i].x *= s.embed_scale, x[i].y *= s.embed_scale, x[i].z *= s.embed_scale, x[i].w *= s.embed_scale;
            }
            if (own)
                for (int k = 0; k < s.n_rot; k++)
                    for (int i = tid; i < s.rot[k].half; i += kNormThreads) {
                        double sn, cs;
                        sincos((double)d.pos[src] * s.rot[k].freq[i], &sn, &cs);
                        s.rot[k].out[(size_t)src * s.rot[k].half + i] = make_float2((float)cs * s.rot[k].mag, (float)sn * s.rot[k].mag);
                    }
        } else {
            const float *xr = a.x + (size_t)src * ldw;
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int j = (tid + i * kNormThreads) * 4;
                x[i] = j < ldw ? load4(xr + j) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
        if (a.y) {
            const AT *yr = reinterpret_cast<const AT *>(a.y) + (size_t)src * ldw, *gr = reinterpret_cast<const AT *>(a.gate) + (size_t)src * a.ldg;
            float4 y[NV];
            float q = 0.f;
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int j = (tid + i * kNormThreads) * 4;
                y[i] = j < ldw ? load4(yr + j) : make_float4(0.f, 0.f, 0.f, 0.f);
                if (a.gate && j < ldw) {
                    const float4 g = load4(gr + j);
                    y[i].x *= sigmoid_act<AT>(g.x), y[i].y *= sigmoid_act<AT>(g.y), y[i].z *= sigmoid_act<AT>(g.z), y[i].w *= sigmoid_act<AT>(g.w);
                }
                q += dot4(y[i]);
            }
            const float f = a.mult / sqrtf(block_sum(q, red) / (float)W + eps);
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int j = (tid + i * kNormThreads) * 4;
                if (j >= ldw) continue;
                const float4 w = load4(a.post + j);
                x[i].x = fmaf(f * y[i].x, w.x, x[i].x), x[i].y = fmaf(f * y[i].y, w.y, x[i].y);
                x[i].z = fmaf(f * y[i].z, w.z, x[i].z), x[i].w = fmaf(f * y[i].w, w.w, x[i].w);
            }
        }
        if (own && a.x_out) {
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int j = (tid + i * kNormThreads) * 4;
                if (j < ldw) store4(a.x_out + (size_t)src * ldw + j, x[i]);
            }
        }
        if (!a.h) continue;
        float q = 0.f;
#pragma unroll
        for (int i = 0; i < NV; i++) q += dot4(x[i]);
        const float f = 1.f / sqrtf(block_sum(q, red) / (float)W + eps);
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int j = (tid + i * kNormThreads) * 4;
            if (j >= ldw) continue;
            const float4 w = load4(a.pre + j);
            x[i].x *= f * w.x, x[i].y *= f * w.y, x[i].z *= f * w.z, x[i].w *= f * w.w;
            if (own) store4(reinterpret_cast<AT *>(a.h) + (size_t)r * ldw + j, x[i]);
        }
        if (!a.shifted) continue;
        if (own) {
            const Seg sg = d.segs[d.ent[r]];
            const bool ok = sg.seq >= 0 && sg.seq < a.max_seqs;
            if (!ok && tid == 0) atomicOr(status, DEV_STATUS_BAD_SEQ);
            float *hist = reinterpret_cast<float *>(a.state + (uint64_t)(ok ? sg.seq : 0) * a.state_stride);
            const bool front = r == sg.row0, last = r == sg.row0 + sg.T - 1;
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int j = (tid + i * kNormThreads) * 4;
                if (j >= ldw) continue;
                float4 b = before[i];
                if (front) b = ok && sg.pos0 > 0 ? load4(hist + (size_t)sg.conv_set * ldw + j) : make_float4(0.f, 0.f, 0.f, 0.f);
                if (last && ok) store4(hist + (size_t)(1 - sg.conv_set) * ldw + j, x[i]);
                const float4 m = load4(a.share + j);
                b.x = fmaf(b.x - x[i].x, m.x, x[i].x), b.y = fmaf(b.y - x[i].y, m.y, x[i].y);
                b.z = fmaf(b.z - x[i].z, m.z, x[i].z), b.w = fmaf(b.w - x[i].w, m.w, x[i].w);
                store4(reinterpret_cast<AT *>(a.shifted) + (size_t)r * ldw + j, b);
            }
        }
#pragma unroll
        for (int i = 0; i < NV; i++) before[i] = x[i];
    }
}

int32_t launch_part_norm(bool f32, const StepDesc &d, const RowSource &embed, const PartNorm &p, const int *rowsel, int rows, float eps, int W, int ldw,
                         int sm_count, int *status, int pdl, cudaStream_t st) {
    const int per = std::max(1, std::min(8, rows / (8 * sm_count)));
    const int nv = (ldw + 4 * kNormThreads - 1) / (4 * kNormThreads);
    JGPT_REQUIRE(nv <= 16, JGPT_ERR_UNSUPPORTED, "width %d", W);
    JGPT_REQUIRE(!p.shifted || !rowsel, JGPT_ERR_INVALID_ARGUMENT, "the token shift takes all rows");
    auto run = [&](auto kern) {
        return launch(kern, (rows + per - 1) / per, 0, pdl, st, (const StepDesc)d, (const RowSource)embed, (const PartNorm)p, rowsel, rows, per, eps, W, ldw, status, pdl);
    };
    auto pick = [&](auto act, auto from_embed) {
        typedef decltype(act) AT;
        constexpr bool E = decltype(from_embed)::value;
        return nv <= 1   ? run(part_norm_kernel<AT, E, 1>)
               : nv <= 2 ? run(part_norm_kernel<AT, E, 2>)
               : nv <= 4 ? run(part_norm_kernel<AT, E, 4>)
               : nv <= 8 ? run(part_norm_kernel<AT, E, 8>)
                         : run(part_norm_kernel<AT, E, 16>);
    };
    if (f32) return p.x ? pick(0.f, std::false_type()) : pick(0.f, std::true_type());
    return p.x ? pick(__nv_bfloat16(), std::false_type()) : pick(__nv_bfloat16(), std::true_type());
}

}  // namespace mix
}  // namespace jgpt
