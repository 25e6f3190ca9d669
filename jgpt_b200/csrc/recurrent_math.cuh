// Elementwise pieces shared by the token-by-token and the chunked form of the recurrent mixers.
#pragma once

#include "mixers.cuh"
#include "ptx.cuh"

namespace jgpt {
namespace mix {

constexpr int kMaxTaps = 8;

__device__ __forceinline__ float2 load2(const __nv_bfloat16 *p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(p)); }
__device__ __forceinline__ float2 load2(const float *p) { return *reinterpret_cast<const float2 *>(p); }
__device__ __forceinline__ float load1(const __nv_bfloat16 *p) { return __bfloat162float(*p); }
__device__ __forceinline__ float load1(const float *p) { return *p; }
__device__ __forceinline__ void store2(__nv_bfloat16 *p, float2 v) { *reinterpret_cast<__nv_bfloat162 *>(p) = __float22bfloat162_rn(v); }
__device__ __forceinline__ void store2(float *p, float2 v) { *reinterpret_cast<float2 *>(p) = v; }
__device__ __forceinline__ void store1(__nv_bfloat16 *p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void store1(float *p, float v) { *p = v; }

// exp for the bf16 mode is the fast one (relative error ~2^-21 on the ranges used here), the exact mode takes expf.
template <class AT>
__device__ __forceinline__ float exp_f(float x) {
    return sizeof(AT) == 4 ? expf(x) : __expf(x);
}
template <class AT>
__device__ __forceinline__ float sigmoid_f(float x) {
    return sizeof(AT) == 4 ? 1.f / (1.f + expf(-x)) : __fdividef(1.f, 1.f + __expf(-x));
}
// log(1 + e^x).  bf16 mode: the fast logarithm; its absolute error (~1e-7, the rounding of a decay near 1) is what counts in
// an exponent.
template <class AT>
__device__ __forceinline__ float softplus_f(float x) {
    return fmaxf(x, 0.f) + (sizeof(AT) == 4 ? log1pf(expf(-fabsf(x))) : __logf(1.f + __expf(-fabsf(x))));
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
    return v;
}

// exp(-exp(y)): the decay of WKV.
template <class AT>
__device__ __forceinline__ float exp_neg_exp(float y) {
    return exp_f<AT>(-exp_f<AT>(y));
}
// Forget gate f = l + (1 - l) sigmoid(z) of HGRN2 and 1 - f = (1 - l) sigmoid(-z), which a difference would round away.
template <class AT>
__device__ __forceinline__ float2 forget_write(float z, float low) {
    return make_float2(low + (1.f - low) * sigmoid_f<AT>(z), (1.f - low) * sigmoid_f<AT>(-z));
}
__host__ __device__ constexpr int rec_key_vectors(int kind) { return kind == REC_GENERAL ? 4 : 3; }  // vectors of key channels per token: q, k, decays, removal
__host__ __device__ constexpr bool rec_has_key(int kind) { return kind != REC_HGRN2; }   // a projection of its own for k
__host__ __device__ constexpr bool rec_has_gate(int kind) { return kind != REC_HGRN2; }  // an output gate
// Gate factor of a head's output from the gate projection.
template <class AT, int KIND>
__device__ __forceinline__ float out_gate(float g) {
    return KIND == REC_DELTA || KIND == REC_GENERAL ? sigmoid_f<AT>(g) : g * sigmoid_f<AT>(g);
}

// RMS norm over a head's value columns and its output gate: raw fp32 values -> activations.  A warp takes heads h0, h0 + 1, ... of a
// row, LANES lanes each with four columns at a time.
template <class AT, int KIND, int LANES>
__device__ __forceinline__ void norm_gate_heads(const RecArgs &a, int r, int h0, int lane) {
    constexpr int NV = LANES == 32 ? 2 : 1;  // up to 256 columns
    const int h = h0 + lane / LANES, c0 = lane % LANES * 4;
    const bool on = h < a.heads;
    const float *raw = a.raw + (size_t)r * a.heads * a.DV + h * a.DV;
    float4 x[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = c0 + 128 * i;
        x[i] = on && c < a.DV ? *reinterpret_cast<const float4 *>(raw + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
    }
    AT *o = reinterpret_cast<AT *>(a.out) + (size_t)r * a.ldo + a.out_off + h * a.DV;
    const AT *gp = KIND == REC_DELTA ? reinterpret_cast<const AT *>(a.z) + (size_t)r * a.ldz + a.zg_off + h * a.DV
                                     : reinterpret_cast<const AT *>(a.proj) + (size_t)r * a.ldp + a.g_off + h * a.DV;
    const float *nw = a.norm_w + h * a.norm_stride;
#pragma unroll
    for (int off = LANES / 2; off >= 1; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    const float inv = a.out_scale / sqrtf(ss / (float)a.vdim + a.eps);
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = c0 + 128 * i;
        if (!on || c >= a.DV) continue;
        const float4 w = *reinterpret_cast<const float4 *>(nw + c);
        float2 lo = make_float2(x[i].x * inv * w.x, x[i].y * inv * w.y), hi = make_float2(x[i].z * inv * w.z, x[i].w * inv * w.w);
        if (rec_has_gate(KIND)) {
            const float2 g0 = load2(gp + c), g1 = load2(gp + c + 2);
            lo.x *= out_gate<AT, KIND>(g0.x), lo.y *= out_gate<AT, KIND>(g0.y), hi.x *= out_gate<AT, KIND>(g1.x), hi.y *= out_gate<AT, KIND>(g1.y);
        }
        store2(o + c, lo), store2(o + c + 2, hi);
    }
}
// Heads a warp takes at once: eight lanes cover 32 columns.
__host__ __device__ inline int norm_heads_per_warp(int DV) { return DV <= 32 ? 4 : (DV <= 64 ? 2 : 1); }
template <class AT, int KIND>
__device__ __forceinline__ void norm_gate_group(const RecArgs &a, int r, int h0, int lane) {
    switch (norm_heads_per_warp(a.DV)) {
        case 4: return norm_gate_heads<AT, KIND, 8>(a, r, h0, lane);
        case 2: return norm_gate_heads<AT, KIND, 16>(a, r, h0, lane);
        default: return norm_gate_heads<AT, KIND, 32>(a, r, h0, lane);
    }
}

}  // namespace mix
}  // namespace jgpt
