// Pieces of the paged attention kernels: activations in either type, page lookup, bf16 products (mma.sync) with fp32 scores and
// weights; the weights enter the second product as a bf16 high and a bf16 low part.
#pragma once

#include "mixers.cuh"
#include "ptx.cuh"

namespace jgpt {
namespace mix {

__device__ __forceinline__ float act_load(const __nv_bfloat16 *p) { return __bfloat162float(*p); }
__device__ __forceinline__ float act_load(const float *p) { return *p; }
__device__ __forceinline__ void act_store(__nv_bfloat16 *p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void act_store(float *p, float v) { *p = v; }

// Physical block of a position, or -1 (recorded in the status word).
template <class Args>
__device__ __forceinline__ int page_of(const Args &a, int seq, int pos) {
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
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t bf16_pair(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t *>(&v);
}
// hi = bf16(x), lo = bf16(x - hi), for two values
__device__ __forceinline__ void split_pair(float x, float y, uint32_t &hi, uint32_t &lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    hi = *reinterpret_cast<const uint32_t *>(&h);
    lo = bf16_pair(x - f.x, y - f.y);
}

// Eight neighbouring elements of an activation row.
__device__ __forceinline__ void load8(const __nv_bfloat16 *p, float (&v)[8]) {
    const uint4 u = *reinterpret_cast<const uint4 *>(p);
    const __nv_bfloat162 *h = reinterpret_cast<const __nv_bfloat162 *>(&u);
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x, v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void load8(const float *p, float (&v)[8]) {
#pragma unroll
    for (int i = 0; i < 8; i += 4) {
        const float4 f = *reinterpret_cast<const float4 *>(p + i);
        v[i] = f.x, v[i + 1] = f.y, v[i + 2] = f.z, v[i + 3] = f.w;
    }
}
__device__ __forceinline__ void store8(__nv_bfloat16 *p, const float (&v)[8]) {
    *reinterpret_cast<uint4 *>(p) = make_uint4(bf16_pair(v[0], v[1]), bf16_pair(v[2], v[3]), bf16_pair(v[4], v[5]), bf16_pair(v[6], v[7]));
}
__device__ __forceinline__ void store8(float *p, const float (&v)[8]) {
    *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]), *reinterpret_cast<float4 *>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

// 16 rows x KT keys of one warp against staged K and V rows: scores, online softmax, P.V.  kat / vat (row, chunk): address of the
// chunk-th 8 elements of a row.  lo / hi: visible key range of this thread's rows g and g + 8 (inclusive),
// with KEEP keys before `keep` are seen as well; kb: first key of the tile.
template <int DK, int DV, int KT, bool KEEP, class QFrag, class KAt, class VAt>
__device__ __forceinline__ void attend_tile(const QFrag &qfrag, const KAt &kat, const VAt &vat, int kb, bool masked, const int (&lo)[2],
                                            const int (&hi)[2], int keep, float scale_log2, float (&m)[2], float (&l)[2], float (&o)[DV / 8][4], int lane) {
    constexpr int NT = KT / 8;
    float s[NT][4];
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) s[j][e] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DK / 16; kk++) {
        uint32_t a[4];
        qfrag(kk, a);
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
            uint32_t b[4];
            ldmatrix_x4(b, kat(j * 8 + ((lane >> 4) << 3) + (lane & 7), kk * 2 + ((lane >> 3) & 1)));
            mma_bf16(s[j], a, b[0], b[1]);
            mma_bf16(s[j + 1], a, b[2], b[3]);
        }
    }
    const int t2 = 2 * (lane & 3);
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int key = kb + j * 8 + t2 + (e & 1), r = e >> 1;
            s[j][e] = (!masked || ((key >= lo[r] || (KEEP && key < keep)) && key <= hi[r])) ? s[j][e] * scale_log2 : -INFINITY;
            mx[r] = fmaxf(mx[r], s[j][e]);
        }
    float f[2];
#pragma unroll
    for (int r = 0; r < 2; r++) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        const float mn = fmaxf(m[r], mx[r]);
        f[r] = mn == -INFINITY ? 1.f : fast_exp2(m[r] - mn);  // nothing visible so far: sums are zero anyway
        m[r] = mn;
        l[r] *= f[r];
    }
    const float mref[2] = {m[0] == -INFINITY ? 0.f : m[0], m[1] == -INFINITY ? 0.f : m[1]};
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            s[j][e] = fast_exp2(s[j][e] - mref[e >> 1]);
            l[e >> 1] += s[j][e];
        }
    if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
        for (int n = 0; n < DV / 8; n++) o[n][0] *= f[0], o[n][1] *= f[0], o[n][2] *= f[1], o[n][3] *= f[1];
    }
#pragma unroll
    for (int kk = 0; kk < KT / 16; kk++) {
        uint32_t ph[4], pl[4];
        split_pair(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
        split_pair(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
        split_pair(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
        split_pair(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
        for (int n = 0; n < DV / 8; n += 2) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, vat(kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), n + (lane >> 4)));
            mma_bf16(o[n], ph, b[0], b[1]);
            mma_bf16(o[n], pl, b[0], b[1]);
            mma_bf16(o[n + 1], ph, b[2], b[3]);
            mma_bf16(o[n + 1], pl, b[2], b[3]);
        }
    }
}

}  // namespace mix
}  // namespace jgpt
