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
__host__ __device__ constexpr bool rec_has_key(int kind) { return kind != REC_HGRN2; }   // a projection of its own for k
__host__ __device__ constexpr bool rec_has_gate(int kind) { return kind != REC_HGRN2; }  // an output gate
// Gate factor of a head's output from the gate projection.
template <class AT, int KIND>
__device__ __forceinline__ float out_gate(float g) {
    return KIND == REC_DELTA ? sigmoid_f<AT>(g) : g * sigmoid_f<AT>(g);
}

// RMS norm over a head's value columns and its output gate, by one warp: raw fp32 values -> activations.
template <class AT, int KIND>
__device__ __forceinline__ void norm_gate_head(const RecArgs &a, int r, int h, int lane) {
    const float *raw = a.raw + (size_t)r * a.heads * a.DV + h * a.DV;
    float ss = 0.f;
    for (int c = lane; c < a.DV; c += 32) ss += raw[c] * raw[c];
    const float inv = a.out_scale / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
    AT *o = reinterpret_cast<AT *>(a.out) + (size_t)r * a.ldo + a.out_off + h * a.DV;
    const AT *gp = KIND == REC_DELTA ? reinterpret_cast<const AT *>(a.z) + (size_t)r * a.ldz + a.zg_off + h * a.DV
                                     : reinterpret_cast<const AT *>(a.proj) + (size_t)r * a.ldp + a.g_off + h * a.DV;
    const float *nw = a.norm_w + h * a.norm_stride;
    for (int c = lane; c < a.DV; c += 32) store1(o + c, raw[c] * inv * nw[c] * (rec_has_gate(KIND) ? out_gate<AT, KIND>(load1(gp + c)) : 1.f));
}

}  // namespace mix
}  // namespace jgpt
