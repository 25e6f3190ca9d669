// The recurrent mixers in chunks of 16 tokens, for long entries of a step.
//
// With the decays of a chunk multiplied up per key channel, b_i = g_1 ... g_i and b_ij = g_{j+1} ... g_i (products of
// factors in (0, 1], never a quotient: nothing overflows however fast a channel decays), the rules
//     GLA    S <- diag(g) S + k v^T                                   o = S^T q
//     DELTA  S <- diag(g) S, u = beta (v - S^T k), S <- S + k u^T     o = S^T q
// become, for a chunk that starts from S0 (GLA: u = v):
//     A_ij = sum_d k_i k_j b_ij  (j < i)      P_ij = sum_d q_i k_j b_ij  (j <= i)
//     u_i + beta_i sum_{j<i} A_ij u_j = beta_i (v_i - (k_i b_i)^T S0)     i.e.  U = T V - (T K~) S0,  T = (I + diag(beta) A)^-1 diag(beta)
//     o_i = (q_i b_i)^T S0 + sum_{j<=i} P_ij u_j
//     S   = diag(b_16) S0 + sum_j (k_j b_16,j) u_j^T
// which follows from unrolling the rules over the chunk.  HGRN2 is GLA with k = 1 - g.  WKV reads before it writes:
//     P_ij = sum_d r_i k_j b_i-1,j  (j < i),  P_ii = sum_d r_i u k_i,  and r_i b_i-1 in place of q_i b_i.
// The generalised delta rule S <- diag(w) S - (a u) (u^T S) + k v^T, with s_i = S_(i-1)^T u_i, is
//     s_i = (u_i b_i-1)^T S0 + sum_{j<i} C_ij v_j - sum_{j<i} A_ij s_j,   A_ij = sum_d u_i (a u)_j b_i-1,j,  C_ij = sum_d u_i k_j b_i-1,j
// so with T = (I + A)^-1 the rows U = -s are  U = -(T U~) S0 - T C V:  the form above with (a u)_j in place of k_j, and the terms
// sum_j (k_j b_16,j) v_j^T of the state and sum_{j<=i} R_ij v_j of the output (R_ij = sum_d q_i k_j b_ij) beside it.
//
// Two kernels.  rec_prep_kernel, parallel over all chunks and heads: convolution, unit vectors, decays, and everything above
// that does not involve S0, written as one record per (chunk, head).  rec_scan_kernel, serial over the chunks of a sequence
// and parallel over heads and 16-column groups of the state: three small products per chunk on the tensor cores
// (mma.sync m16n8k8, every fp32 operand as a TF32 high and low part: three products, fp32-level accuracy).  A warp holds S^T
// of its 16 value columns as fp32 accumulators; the accumulator layout IS the A operand layout of the next chunk once channels
// 2t, 2t+1 of a k step are taken in the order (t, t + 4), so the state never leaves registers.  Records come in by bulk copies.
#include <algorithm>
#include <type_traits>

#include "recurrent_math.cuh"

namespace jgpt {
namespace mix {

constexpr int kC = kRecChunk;
static_assert(kC == 16, "the layouts below are for 16 tokens");

// Record of one (chunk, head), floats:
//   [DELTA: -W [16 tok][DK]] [Q~ [16 tok][DK]] [K^ [DK][16 tok]] [b_16 [DK]] [P [16 i][16 j]] [U0 [DV][16 tok]]
// GENERAL: -W, Q~, K^ with (a u), K^ with k, b_16, P with (a u), R, then for every 16 value columns U0 [16][16 tok] and V [16][16 tok].
// 8-float groups inside a row are permuted so that the fragment loads are free of bank conflicts.
__host__ __device__ constexpr int rec_mats(int kind) { return kind == REC_GENERAL ? 4 : kind == REC_DELTA ? 3 : 2; }
__host__ __device__ constexpr int rec_updates(int kind) { return kind == REC_GENERAL ? 2 : 1; }  // outer products per token
__host__ __device__ constexpr bool rec_has_w(int kind) { return kind == REC_DELTA || kind == REC_GENERAL; }
__host__ __device__ constexpr uint64_t record_floats(int kind, int DK, int DV) {
    return (uint64_t)rec_mats(kind) * kC * DK + DK + (uint64_t)rec_updates(kind) * (kC * kC + kC * (uint64_t)DV);
}
uint64_t rec_chunk_record_floats(int kind, int DK, int DV) { return record_floats(kind, DK, DV); }
int rec_chunk_min_tokens(bool f32) {
    if (f32 && !env_int("JGPT_B200_REC_CHUNK_EXACT", 0)) return 0;  // the exact mode stays token by token
    return std::max(0, env_int("JGPT_B200_REC_CHUNK_MIN", 32));
}
// [token][channel] rows: 8-groups xor token & 3.  [x][16] rows: the two 8-groups swapped when bit 1 of x is set.
__device__ __forceinline__ int at_tok(int tok, int ch, int DK) { return tok * DK + ((((ch >> 3) ^ (tok & 3)) << 3) | (ch & 7)); }
__device__ __forceinline__ int at_16(int x, int j) { return x * 16 + ((((j >> 3) ^ ((x >> 1) & 1)) << 3) | (j & 7)); }

__device__ __forceinline__ void store_row16(float *m, int x, const float (&v)[16]) {
#pragma unroll
    for (int j = 0; j < 16; j += 4) *reinterpret_cast<float4 *>(m + at_16(x, j)) = make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]);
}

// Row i of a lower triangular 16 x 16 matrix in shared memory times x (entries past i are not touched).
__device__ __forceinline__ float lower_dot(const float *T, int i, const float (&x)[16]) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < 16; j += 4)
        if (j <= i) {
            const float4 q = *reinterpret_cast<const float4 *>(T + i * 16 + j);
            s = fmaf(q.x, x[j], s);
            if (j + 1 <= i) s = fmaf(q.y, x[j + 1], s);
            if (j + 2 <= i) s = fmaf(q.z, x[j + 2], s);
            if (j + 3 <= i) s = fmaf(q.w, x[j + 3], s);
        }
    return s;
}

// 32 sums over the 32 lanes: lane L returns the total of v[L].
__device__ __forceinline__ float reduce32(float (&v)[32], int lane) {
#pragma unroll
    for (int n = 16; n >= 1; n >>= 1) {
        const bool up = lane & n;
#pragma unroll
        for (int i = 0; i < 16; i++)
            if (i < n) v[i] = (up ? v[i + n] : v[i]) + __shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + n], n);
    }
    return v[0];
}

template <class AT, int KIND, int DK>
__global__ void __launch_bounds__(256) rec_prep_kernel(const RecArgs a, const Seg *__restrict__ segs, const int2 *__restrict__ chunks, int pdl) {
    constexpr int NI = DK / 32;
    extern __shared__ __align__(16) float prep_smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, DV = a.DV;
    float *sq = prep_smem, *sk = sq + kC * DK, *sg = sk + kC * DK, *sv = sg + kC * DK;  // [16][DK], [16][DV]
    float *sA = sv + kC * DV, *sP = sA + kC * kC, *sT = sP + kC * kC, *sbeta = sT + kC * kC;
    float *sR = sbeta + kC, *sC = sR + kC * kC, *sa = sC + kC * kC;  // general
    if (pdl & 2) griddep_launch_dependents();
    const int2 ck = chunks[blockIdx.x];
    const Seg sgm = segs[ck.x];
    const int t0 = ck.y, tn = min(kC, sgm.T - t0);
    if (sgm.seq < 0 || sgm.seq >= a.max_seqs) return;  // the scan reports it
    if (pdl & 1) griddep_wait();

    const AT *__restrict__ proj = reinterpret_cast<const AT *>(a.proj) + (size_t)sgm.row0 * a.ldp;
    const AT *__restrict__ z = reinterpret_cast<const AT *>(a.z) + (size_t)sgm.row0 * a.ldz;
    uint8_t *part = a.state + (uint64_t)sgm.seq * a.state_stride;
    const int kvh = h / (a.heads / a.kv_heads), nq = a.kv_heads * DK, channels = 2 * nq + a.heads * DV;
    const AT *hist = reinterpret_cast<const AT *>(part + a.conv_off) + (size_t)sgm.conv_set * (a.taps > 0 ? a.taps - 1 : 0) * channels;
    const float qscale = rsqrtf((float)a.dim), rate = KIND == REC_DELTA ? expf(a.a_log[h]) : 1.f / a.tau;
    auto conv_input = [&](int t, int pc, int ch) -> float2 {
        if (t >= 0) return load2(proj + (size_t)t * a.ldp + pc);
        if (sgm.pos0 + t >= 0) return load2(hist + (size_t)(-1 - t) * channels + ch);
        return make_float2(0.f, 0.f);
    };
    auto locate = [&](int idx, int &pc, int &ch) {
        if (idx < DK) {
            const bool is_k = idx >= DK / 2;
            const int c = kvh * DK + 2 * idx - (is_k ? DK : 0);
            pc = (is_k ? a.k_off : a.q_off) + c, ch = (is_k ? nq : 0) + c;
        } else {
            const int c = h * DV + 2 * (idx - DK);
            pc = a.v_off + c, ch = 2 * nq + c;
        }
    };
    const int npairs = DK + DV / 2;
    // decay logits and step sizes are requested first and used last
    constexpr int ZN = (kC * DK / 2 + 255) / 256;
    float2 zr[ZN];
#pragma unroll
    for (int e = 0; e < ZN; e++) {
        const int idx = e * 256 + tid, t = idx / (DK / 2), c = 2 * (idx % (DK / 2));
        zr[e] = t < tn ? load2(z + (size_t)(t0 + t) * a.ldz + a.z_off + h * DK + c) : make_float2(0.f, 0.f);
        if (KIND == REC_GENERAL && t < kC) {
            float2 m = make_float2(0.f, 0.f);
            if (t < tn) {
                const float2 mb = *reinterpret_cast<const float2 *>(a.removal_bias + h * DK + c);
                m = load2(proj + (size_t)(t0 + t) * a.ldp + a.b_off + h * DK + c);
                m.x = sigmoid_f<AT>(m.x + mb.x), m.y = sigmoid_f<AT>(m.y + mb.y);
            }
            *reinterpret_cast<float2 *>(sa + t * DK + c) = m;
        }
    }
    float bl = 0.f;
    if (KIND == REC_DELTA && tid < tn) bl = load1(proj + (size_t)(t0 + tid) * a.ldp + a.b_off + h);
    // ---- q, k, v of the chunk ----
    auto convolve = [&](auto max_taps, int pc, int ch, float *dst, int ld) {
        constexpr int MT = decltype(max_taps)::value;
        const float *w = (ch < nq ? a.conv_q + (size_t)ch * a.taps
                                  : (ch < 2 * nq ? a.conv_k + (size_t)(ch - nq) * a.taps : a.conv_v + (size_t)(ch - 2 * nq) * a.taps));
        float2 wt[MT], x[kC + MT - 1];  // x[i]: token t0 + i - (MT - 1); every load in flight at once
#pragma unroll
        for (int back = 0; back < MT; back++) wt[back] = back < a.taps ? make_float2(w[a.taps - 1 - back], w[2 * a.taps - 1 - back]) : make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < kC + MT - 1; i++) {
            const int t = t0 + i - (MT - 1);
            x[i] = i < MT - 1 ? (MT - 1 - i < a.taps ? conv_input(t, pc, ch) : make_float2(0.f, 0.f))
                              : (i - (MT - 1) < tn ? load2(proj + (size_t)t * a.ldp + pc) : make_float2(0.f, 0.f));
        }
#pragma unroll
        for (int t = 0; t < kC; t++) {
            float2 y = make_float2(0.f, 0.f);
#pragma unroll
            for (int back = 0; back < MT; back++) y.x = fmaf(wt[back].x, x[t + MT - 1 - back].x, y.x), y.y = fmaf(wt[back].y, x[t + MT - 1 - back].y, y.y);
            *reinterpret_cast<float2 *>(dst + t * ld) = t < tn ? make_float2(y.x * sigmoid_f<AT>(y.x), y.y * sigmoid_f<AT>(y.y)) : make_float2(0.f, 0.f);
        }
    };
    for (int idx = tid; idx < npairs; idx += 256) {
        int pc, ch;
        locate(idx, pc, ch);
        float *dst = idx < DK / 2 ? sq + 2 * idx : (idx < DK ? sk + 2 * idx - DK : sv + 2 * (idx - DK));
        const int ld = idx < DK ? DK : DV;
        if (KIND == REC_DELTA) {
            if (a.taps <= 4) convolve(std::integral_constant<int, 4>(), pc, ch, dst, ld);
            else convolve(std::integral_constant<int, kMaxTaps>(), pc, ch, dst, ld);
        } else {
            if (!rec_has_key(KIND) && idx >= DK / 2 && idx < DK) continue;  // its key comes with the forget gate
            float2 x[kC];
            const float f = KIND == REC_GLA && idx < DK / 2 ? qscale : 1.f;
#pragma unroll
            for (int t = 0; t < kC; t++) x[t] = t < tn ? load2(proj + (size_t)(t0 + t) * a.ldp + pc) : make_float2(0.f, 0.f);
#pragma unroll
            for (int t = 0; t < kC; t++) {
                if (KIND == REC_HGRN2 && idx < DK / 2) x[t].x *= sigmoid_f<AT>(x[t].x), x[t].y *= sigmoid_f<AT>(x[t].y);
                else x[t].x *= f, x[t].y *= f;
                *reinterpret_cast<float2 *>(dst + t * ld) = x[t];
            }
        }
    }
    // ---- decays (1 past the end: the state stays) and step sizes ----
#pragma unroll
    for (int e = 0; e < ZN; e++) {
        const int idx = e * 256 + tid, t = idx / (DK / 2), c = 2 * (idx % (DK / 2));
        if (t >= kC) break;
        float2 y = make_float2(1.f, 1.f), w = make_float2(0.f, 0.f);
        if (t < tn) {
            const float2 b = *reinterpret_cast<const float2 *>(a.decay_bias + h * DK + c);
            y.x = zr[e].x + b.x, y.y = zr[e].y + b.y;
            if (KIND == REC_GLA) y.x = -y.x, y.y = -y.y;
            if (KIND == REC_HGRN2) {
                const float2 low = *reinterpret_cast<const float2 *>(a.lower + h * DK + c);
                const float2 f0 = forget_write<AT>(y.x, low.x), f1 = forget_write<AT>(y.y, low.y);
                y = make_float2(f0.x, f1.x), w = make_float2(f0.y, f1.y);
            } else if (KIND == REC_WKV) {
                y.x = exp_neg_exp<AT>(y.x), y.y = exp_neg_exp<AT>(y.y);
            } else if (KIND == REC_GENERAL) {
                y.x = exp_f<AT>(-a.rate * sigmoid_f<AT>(y.x)), y.y = exp_f<AT>(-a.rate * sigmoid_f<AT>(y.y));
            } else {
                y.x = exp_f<AT>(-rate * softplus_f<AT>(y.x)), y.y = exp_f<AT>(-rate * softplus_f<AT>(y.y));
            }
        }
        if (KIND == REC_HGRN2) *reinterpret_cast<float2 *>(sk + t * DK + c) = w;
        *reinterpret_cast<float2 *>(sg + t * DK + c) = y;
    }
    if (KIND == REC_DELTA && tid < kC) sbeta[tid] = tid < tn ? sigmoid_f<AT>(bl) : 0.f;
    __syncthreads();
    if (KIND == REC_DELTA) {
        for (int t = warp; t < kC; t += 8) {
            float qv[NI], kv[NI], qq = 0.f, kk = 0.f;
#pragma unroll
            for (int i = 0; i < NI; i++) {
                qv[i] = sq[t * DK + lane + 32 * i], kv[i] = sk[t * DK + lane + 32 * i];
                qq += qv[i] * qv[i], kk += kv[i] * kv[i];
            }
            const float fq = qscale / sqrtf(warp_sum(qq) + 1e-6f), fk = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
#pragma unroll
            for (int i = 0; i < NI; i++) sq[t * DK + lane + 32 * i] = qv[i] * fq, sk[t * DK + lane + 32 * i] = kv[i] * fk;
        }
        __syncthreads();
    }
    if (KIND == REC_GENERAL) {  // |k| beside the unit key, which the removal rates are multiplied with
        for (int t = warp; t < kC; t += 8) {
            float kv[NI], kk = 0.f;
#pragma unroll
            for (int i = 0; i < NI; i++) kv[i] = sk[t * DK + lane + 32 * i], kk += kv[i] * kv[i];
            const float n = sqrtf(warp_sum(kk) + 1e-6f), f = 1.f / n;
#pragma unroll
            for (int i = 0; i < NI; i++) sk[t * DK + lane + 32 * i] = kv[i] * f, sa[t * DK + lane + 32 * i] *= kv[i] * f;
            if (lane == 0) sbeta[t] = n;
        }
        __syncthreads();
    }
    // ---- A and P: warp w takes keys j = w and 15 - w; the key decays step by step on its way to later tokens ----
    {
        const int js[2] = {warp, 15 - warp};
        float v[2][32], bonus[NI];
        if (KIND == REC_WKV) {
#pragma unroll
            for (int c = 0; c < NI; c++) bonus[c] = a.bonus[h * DK + lane + 32 * c];
        }
        if (KIND == REC_GENERAL) {
#pragma unroll 1
            for (int s = 0; s < 2; s++) {
                const int j = js[s];
                const float n = sbeta[j];
                float kd[NI], ad[NI], w[2][32];  // unit key and removal row on their way; rows P, A and R, C
#pragma unroll
                for (int c = 0; c < NI; c++) kd[c] = sk[j * DK + lane + 32 * c], ad[c] = sa[j * DK + lane + 32 * c];
#pragma unroll
                for (int i = 0; i < kC; i++) {
                    float p = 0.f, x = 0.f, y = 0.f, z = 0.f;
                    if (i >= j) {
#pragma unroll
                        for (int c = 0; c < NI; c++) {
                            if (i > j) {
                                const float u = sk[i * DK + lane + 32 * c], g = sg[i * DK + lane + 32 * c];
                                x = fmaf(u, ad[c], x), z = fmaf(u, kd[c], z);
                                ad[c] *= g, kd[c] *= g;
                            }
                            const float q = sq[i * DK + lane + 32 * c];
                            p = fmaf(q, ad[c], p), y = fmaf(q, kd[c], y);
                        }
                    }
                    w[0][i] = p, w[0][16 + i] = x, w[1][i] = y, w[1][16 + i] = z;
                }
                const float t0 = reduce32(w[0], lane), t1 = n * reduce32(w[1], lane);
                if (lane < 16) sP[lane * kC + j] = t0, sR[lane * kC + j] = t1;
                else sA[(lane - 16) * kC + j] = t0, sC[(lane - 16) * kC + j] = t1;
            }
        }
#pragma unroll
        for (int s = 0; s < (KIND == REC_GENERAL ? 0 : 2); s++) {
            const int j = js[s];
            float kk[NI];
#pragma unroll
            for (int c = 0; c < NI; c++) kk[c] = sk[j * DK + lane + 32 * c];
#pragma unroll
            for (int i = 0; i < kC; i++) {
                float p = 0.f, w = 0.f;
                if (i >= j) {
#pragma unroll
                    for (int c = 0; c < NI; c++) {
                        if (KIND == REC_WKV) {  // the bonus for itself, undecayed for the next token
                            p = fmaf(sq[i * DK + lane + 32 * c], i == j ? kk[c] * bonus[c] : kk[c], p);
                            if (i > j) kk[c] *= sg[i * DK + lane + 32 * c];
                            continue;
                        }
                        if (i > j) kk[c] *= sg[i * DK + lane + 32 * c];
                        p = fmaf(sq[i * DK + lane + 32 * c], kk[c], p);
                        if (KIND == REC_DELTA) w = fmaf(sk[i * DK + lane + 32 * c], kk[c], w);
                    }
                }
                if (KIND == REC_DELTA) v[s][i] = p, v[s][16 + i] = i > j ? w : 0.f;
                else v[0][16 * s + i] = p;
            }
            if (KIND == REC_DELTA) {
                const float tot = reduce32(v[s], lane);
                if (lane < 16) sP[lane * kC + j] = tot;
                else sA[(lane - 16) * kC + j] = tot;
            }
        }
        if (KIND != REC_DELTA && KIND != REC_GENERAL) {
            const float tot = reduce32(v[0], lane);
            sP[(lane & 15) * kC + js[lane >> 4]] = tot;
        }
    }
    __syncthreads();
    if (rec_has_w(KIND) && tid < kC) {  // column tid of T by forward substitution
        float t[kC];
#pragma unroll
        for (int i = 0; i < kC; i++) {
            float s = i == tid ? 1.f : 0.f;
#pragma unroll
            for (int j = 0; j < kC; j++)
                if (j < i) s = fmaf(-sA[i * kC + j], t[j], s);
            t[i] = KIND == REC_DELTA ? sbeta[i] * s : s;
            sT[i * kC + tid] = t[i];
        }
    }
    if (rec_has_w(KIND)) __syncthreads();
    // ---- the record ----
    float *rec = a.chunk_ws + ((size_t)blockIdx.x * a.heads + h) * record_floats(KIND, DK, DV);
    float *rw = rec, *rq = rec + (rec_has_w(KIND) ? kC * DK : 0), *rk = rq + kC * DK, *rb = rk + rec_updates(KIND) * kC * DK, *rp = rb + DK,
          *ru = rp + rec_updates(KIND) * kC * kC;
    for (int idx = tid; idx < DK + DV; idx += 256) {
        if (idx < DK) {
            const int d = idx;
            float kt[kC], b = 1.f;
#pragma unroll
            for (int t = 0; t < kC; t++) {
                if (KIND == REC_WKV) rq[at_tok(t, d, DK)] = sq[t * DK + d] * b;
                if (KIND == REC_GENERAL) kt[t] = sk[t * DK + d] * b;
                b *= sg[t * DK + d];
                if (KIND != REC_WKV) rq[at_tok(t, d, DK)] = sq[t * DK + d] * b;
                if (KIND != REC_GENERAL) kt[t] = sk[t * DK + d] * b;
            }
            rb[d] = b;
            if (rec_has_w(KIND)) {
#pragma unroll
                for (int i = 0; i < kC; i++) {
                    rw[at_tok(i, d, DK)] = -lower_dot(sT, i, kt);
                }
            }
            b = 1.f;
#pragma unroll
            for (int t = kC - 1; t >= 0; t--) {
                kt[t] = (KIND == REC_GENERAL ? sa : sk)[t * DK + d] * b;
                b *= sg[t * DK + d];
            }
            store_row16(rk, d, kt);
            if (KIND == REC_GENERAL) {
                b = 1.f;
#pragma unroll
                for (int t = kC - 1; t >= 0; t--) {
                    kt[t] = sbeta[t] * sk[t * DK + d] * b;
                    b *= sg[t * DK + d];
                }
                store_row16(rk + kC * DK, d, kt);
            }
        } else {
            const int c = idx - DK;
            float vv[kC];
#pragma unroll
            for (int t = 0; t < kC; t++) vv[t] = sv[t * DV + c];
            if (KIND == REC_DELTA) {
#pragma unroll
                for (int i = kC - 1; i >= 0; i--) {  // T is lower triangular: row i needs rows up to i only
                    vv[i] = lower_dot(sT, i, vv);
                }
            }
            if (KIND == REC_GENERAL) {  // V, then -T C V; C is strictly lower triangular
                float *cols = ru + c / 16 * (2 * 16 * kC);
                store_row16(cols + 16 * kC, c % 16, vv);
#pragma unroll
                for (int i = kC - 1; i >= 0; i--) vv[i] = lower_dot(sC, i, vv);
#pragma unroll
                for (int i = kC - 1; i >= 0; i--) vv[i] = -lower_dot(sT, i, vv);
                store_row16(cols, c % 16, vv);
                continue;
            }
            store_row16(ru, c, vv);
        }
    }
    for (int e = tid; e < kC * kC; e += 256) {
        rp[at_16(e / kC, e % kC)] = e / kC >= e % kC ? sP[e] : 0.f;
        if (KIND == REC_GENERAL) rp[kC * kC + at_16(e / kC, e % kC)] = e / kC >= e % kC ? sR[e] : 0.f;
    }
    // ---- convolution history for the next step, by the entry's last chunk ----
    if (KIND == REC_DELTA && a.taps > 1 && t0 + kC >= sgm.T) {
        AT *next = reinterpret_cast<AT *>(part + a.conv_off) + (size_t)(1 - sgm.conv_set) * (a.taps - 1) * channels;
        const bool first_of_group = h % (a.heads / a.kv_heads) == 0;
        for (int idx = tid; idx < npairs; idx += 256) {
            if (idx < DK && !first_of_group) continue;  // shared channels are written once
            int pc, ch;
            locate(idx, pc, ch);
            for (int i = 0; i < a.taps - 1; i++) store2(next + (size_t)i * channels + ch, conv_input(sgm.T - 1 - i, pc, ch));
        }
    }
}

// TF32 high and low part by truncation (the remainder is exact before its own truncation: ~2^-21 together).  Two masks and
// a subtraction; the rounding conversion would give half a bit more and costs the scan more issue time than its products.
__device__ __forceinline__ void split_trunc(float x, uint32_t &hi, uint32_t &lo) {
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi)) & 0xffffe000u;
}
// hi / lo TF32 parts of an A fragment held as accumulators (see the order note above) and the three-product update.
struct SplitA {
    uint32_t hi[4], lo[4];
    __device__ __forceinline__ explicit SplitA(const float (&c)[4]) {
        split_trunc(c[0], hi[0], lo[0]), split_trunc(c[2], hi[1], lo[1]), split_trunc(c[1], hi[2], lo[2]), split_trunc(c[3], hi[3], lo[3]);
    }
};
struct SplitB {
    uint32_t hi[2], lo[2];
    __device__ __forceinline__ explicit SplitB(const float2 v) { split_trunc(v.x, hi[0], lo[0]), split_trunc(v.y, hi[1], lo[1]); }
};
__device__ __forceinline__ void mma3(float (&acc)[4], float (&cor)[4], const SplitA &x, const SplitB &y) {
    mma_tf32(cor, x.lo, y.hi[0], y.hi[1]);
    mma_tf32(acc, x.hi, y.hi[0], y.hi[1]);
    mma_tf32(cor, x.hi, y.lo[0], y.lo[1]);
}

// Two stages where three do not fit beside one another.
__host__ __device__ constexpr int scan_stages(int kind, int DK) { return kind == REC_GENERAL && DK > 192 ? 2 : 3; }
__host__ __device__ constexpr size_t scan_stage_floats(int kind, int DK, int cols) { return (size_t)record_floats(kind, DK, cols); }

template <int KIND, int DK>
__global__ void __launch_bounds__(256) rec_scan_kernel(const RecArgs a, const Seg *__restrict__ segs, const int2 *__restrict__ longs, int pdl) {
    constexpr int NT = DK / 8;
    constexpr int UPD = rec_updates(KIND), kScanStages = scan_stages(KIND, DK);
    constexpr uint32_t COMMON = (uint32_t)(rec_mats(KIND) * kC * DK + DK + UPD * kC * kC);
    extern __shared__ __align__(16) float scan_smem[];
    __shared__ __align__(8) uint64_t full[kScanStages];
    __shared__ int s_abort_mem;
    volatile int *s_abort = &s_abort_mem;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int cols = blockDim.x / 2, h = blockIdx.x % a.heads, col0 = blockIdx.x / a.heads * cols;  // value columns of this CTA
    const uint32_t STAGE = COMMON + (uint32_t)(UPD * kC) * cols;
    if (pdl & 2) griddep_launch_dependents();
    const int2 ls = longs[blockIdx.y];
    const Seg sgm = segs[ls.x];
    if (sgm.seq < 0 || sgm.seq >= a.max_seqs) {
        if (tid == 0) atomicOr(a.status, DEV_STATUS_BAD_SEQ);
        return;
    }
    if (tid == 0) {
        for (int s = 0; s < kScanStages; s++) mbar_init(&full[s], 1);
        *s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    float *S = reinterpret_cast<float *>(a.state + (uint64_t)sgm.seq * a.state_stride) + ((size_t)h * (a.DV / 16) + col0 / 16 + warp) * (DK * 16);
    float st[NT][4];  // (column g, channel 8 n + 2 t), (g, + 1), (g + 8, ..), (g + 8, + 1)
#pragma unroll
    for (int n = 0; n < NT; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) st[n][e] = sgm.pos0 > 0 ? S[(size_t)(8 * n + 2 * t + (e & 1)) * 16 + g + 8 * (e >> 1)] : 0.f;
    __syncthreads();
    if (pdl & 1) griddep_wait();

    const int n_chunks = (sgm.T + kC - 1) / kC;
    const uint64_t rec_floats = record_floats(KIND, DK, a.DV);
    const float *rec0 = a.chunk_ws + ((size_t)ls.y * a.heads + h) * rec_floats;
    auto fetch = [&](int c) {  // one thread
        const int s = c % kScanStages;
        const float *rec = rec0 + (size_t)c * a.heads * rec_floats;
        float *dst = scan_smem + (size_t)s * STAGE;
        mbar_expect_tx(&full[s], STAGE * 4);
        bulk_g2s(dst, rec, COMMON * 4, &full[s]);
        bulk_g2s(dst + COMMON, rec + COMMON + (size_t)(UPD * kC) * col0, (uint32_t)(UPD * kC * cols * 4), &full[s]);
    };
    int issued = 0;
    if (tid == 0)
        for (; issued < kScanStages && issued < n_chunks; issued++) fetch(issued);
    for (int c = 0; c < n_chunks; c++) {
        const int s = c % kScanStages;
        const bool ok = mbar_wait_bounded(&full[s], (uint32_t)(c / kScanStages) & 1u, a.status, s_abort);
        if (__syncthreads_or(!ok)) {  // give copies in flight a bounded chance to land, then leave together
            if (tid == 0)
                for (int k = c; k < issued; k++)
                    for (uint32_t i = 0; i < (1u << 16) && !mbar_try_wait(&full[k % kScanStages], (uint32_t)(k / kScanStages) & 1u); i++) {
                    }
            __syncthreads();
            return;
        }
        const float *m = scan_smem + (size_t)s * STAGE;
        const float *mw = m, *mq = m + (rec_has_w(KIND) ? kC * DK : 0), *mk = mq + kC * DK, *mb = mk + UPD * kC * DK, *mp = mb + DK,
                    *mu = m + COMMON + (size_t)warp * 16 * UPD * kC;
        // U0 and O, tokens 8 n + 2 t (+ 1) of columns g, g + 8
        float u[2][4], uc[2][4], o[2][4], oc[2][4];
#pragma unroll
        for (int n = 0; n < 2; n++) {
            const float2 x = *reinterpret_cast<const float2 *>(mu + at_16(g, 8 * n + 2 * t)), y = *reinterpret_cast<const float2 *>(mu + at_16(g + 8, 8 * n + 2 * t));
            u[n][0] = x.x, u[n][1] = x.y, u[n][2] = y.x, u[n][3] = y.y;
#pragma unroll
            for (int e = 0; e < 4; e++) uc[n][e] = o[n][e] = oc[n][e] = 0.f;
        }
#pragma unroll
        for (int k = 0; k < NT; k++) {
            const SplitA sa(st[k]);
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const int at = at_tok(8 * n + g, 8 * k + 2 * t, DK);
                if (rec_has_w(KIND)) mma3(u[n], uc[n], sa, SplitB(*reinterpret_cast<const float2 *>(mw + at)));
                mma3(o[n], oc[n], sa, SplitB(*reinterpret_cast<const float2 *>(mq + at)));
            }
        }
        if (rec_has_w(KIND)) {
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) u[n][e] += uc[n][e];
        }
        const SplitA ua[2] = {SplitA(u[0]), SplitA(u[1])};
        if (KIND == REC_GENERAL) {  // V takes the place of U0 for the second set of products
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const float *mv = mu + 16 * kC;
                const float2 x = *reinterpret_cast<const float2 *>(mv + at_16(g, 8 * n + 2 * t)), y = *reinterpret_cast<const float2 *>(mv + at_16(g + 8, 8 * n + 2 * t));
                u[n][0] = x.x, u[n][1] = x.y, u[n][2] = y.x, u[n][3] = y.y;
            }
        }
        const SplitA va[2] = {SplitA(u[0]), SplitA(u[1])};
#pragma unroll
        for (int k = 0; k < 2; k++)
#pragma unroll
            for (int n = 0; n < 2; n++) {
                mma3(o[n], oc[n], ua[k], SplitB(*reinterpret_cast<const float2 *>(mp + at_16(8 * n + g, 8 * k + 2 * t))));
                if (KIND == REC_GENERAL) mma3(o[n], oc[n], va[k], SplitB(*reinterpret_cast<const float2 *>(mp + kC * kC + at_16(8 * n + g, 8 * k + 2 * t))));
            }
        // the state moves on
#pragma unroll
        for (int n = 0; n < NT; n++) {
            const float2 b = *reinterpret_cast<const float2 *>(mb + 8 * n + 2 * t);
            float cor[4] = {0.f, 0.f, 0.f, 0.f};
            st[n][0] *= b.x, st[n][1] *= b.y, st[n][2] *= b.x, st[n][3] *= b.y;
#pragma unroll
            for (int k = 0; k < 2; k++) {
                mma3(st[n], cor, ua[k], SplitB(*reinterpret_cast<const float2 *>(mk + at_16(8 * n + g, 8 * k + 2 * t))));
                if (KIND == REC_GENERAL) mma3(st[n], cor, va[k], SplitB(*reinterpret_cast<const float2 *>(mk + kC * DK + at_16(8 * n + g, 8 * k + 2 * t))));
            }
#pragma unroll
            for (int e = 0; e < 4; e++) st[n][e] += cor[e];
        }
        float *raw = a.raw + (size_t)(sgm.row0 + c * kC) * (a.heads * a.DV) + h * a.DV + col0 + warp * 16;
        const int tn = sgm.T - c * kC;
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int tok = 8 * n + 2 * t + (e & 1);
                if (tok < tn) raw[(size_t)tok * (a.heads * a.DV) + g + 8 * (e >> 1)] = o[n][e] + oc[n][e];
            }
        __syncthreads();  // everyone is done with the stage
        if (tid == 0 && issued < n_chunks) fetch(issued++);
    }
#pragma unroll
    for (int n = 0; n < NT; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) S[(size_t)(8 * n + 2 * t + (e & 1)) * 16 + g + 8 * (e >> 1)] = st[n][e];
}

// RMS norm and gate of the chunked rows.
template <class AT, int KIND>
__global__ void __launch_bounds__(256) rec_chunk_norm_kernel(const RecArgs a, const Seg *__restrict__ segs, const int2 *__restrict__ chunks, int pdl) {
    if (pdl & 2) griddep_launch_dependents();
    const int2 ck = chunks[blockIdx.x];
    const Seg sgm = segs[ck.x];
    const int tn = min(kC, sgm.T - ck.y), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (pdl & 1) griddep_wait();
    const int per = norm_heads_per_warp(a.DV), groups = (a.heads + per - 1) / per;
    for (int i = blockIdx.y * 8 + warp; i < tn * groups; i += 8 * gridDim.y)
        norm_gate_group<AT, KIND>(a, sgm.row0 + ck.y + i / groups, i % groups * per, lane);
}

template <class K, class... Args>
static int32_t launch_early(K kern, dim3 grid, int threads, size_t smem, int &set_for, size_t smem_max, int pdl, cudaStream_t st, Args... args) {
    int dev = 0;
    JGPT_CUDA_TRY(cudaGetDevice(&dev));
    if (set_for != dev) {
        if (smem_max > 48 * 1024) JGPT_CUDA_TRY(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_max));
        set_for = dev;
    }
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = grid, cfg.blockDim = dim3((unsigned)threads), cfg.dynamicSmemBytes = smem, cfg.stream = st;
    cfg.attrs = attr, cfg.numAttrs = (pdl & 1) ? 1 : 0;
    JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, kern, args...));
    return JGPT_OK;
}

template <class AT, int KIND, int DK>
static int32_t chunk_launch(const StepDesc &d, const RecArgs &a, int pdl, cudaStream_t st) {
    JGPT_REQUIRE((uint64_t)d.n_chunks * a.heads * record_floats(KIND, DK, a.DV) <= a.chunk_ws_floats, JGPT_ERR_INVALID_ARGUMENT,
                 "%d chunks exceed the workspace", d.n_chunks);
    auto prep_smem = [](int DV) { return sizeof(float) * ((size_t)kC * (rec_key_vectors(KIND) * DK + DV) + (KIND == REC_GENERAL ? 5 : 3) * kC * kC + kC); };
    static thread_local int set1 = -1, set2 = -1, set3 = -1;
    int32_t rc = launch_early(rec_prep_kernel<AT, KIND, DK>, dim3((unsigned)d.n_chunks, (unsigned)a.heads), 256, prep_smem(a.DV), set1, prep_smem(256), pdl,
                              st, a, d.segs, d.chunks, pdl);
    if (rc) return rc;
    // warps (16 value columns each) per CTA: as many as still leave every SM a CTA
    const int groups = a.DV / 16, max_warps = DK <= 128 ? 8 : 4;
    int nw = std::min(groups, max_warps);
    while (nw > 1 && (groups % nw != 0 || (long long)a.heads * d.n_long * (groups / nw) < a.sm_count)) nw--;
    constexpr int form = rec_has_w(KIND) ? KIND : REC_GLA, stages = scan_stages(form, DK);
    const size_t smem = sizeof(float) * stages * scan_stage_floats(KIND, DK, 16 * nw);
    rc = launch_early(rec_scan_kernel<form, DK>, dim3((unsigned)(a.heads * (groups / nw)), (unsigned)d.n_long), 32 * nw, smem, set2,
                      sizeof(float) * stages * scan_stage_floats(KIND, DK, 16 * max_warps), pdl, st, a, d.segs, d.long_segs, pdl);
    if (rc) return rc;
    return launch_early(rec_chunk_norm_kernel<AT, KIND>, dim3((unsigned)d.n_chunks, (unsigned)((kC * (a.heads / norm_heads_per_warp(a.DV) + 1) + 31) / 32)), 256, 0, set3, 0, pdl, st, a, d.segs,
                        d.chunks, pdl);
}

template <class AT, int KIND>
static int32_t chunk_dispatch(const StepDesc &d, const RecArgs &a, int pdl, cudaStream_t st) {
    switch (a.DK) {
        case 32: return chunk_launch<AT, KIND, 32>(d, a, pdl, st);
        case 64: return chunk_launch<AT, KIND, 64>(d, a, pdl, st);
        case 96: return chunk_launch<AT, KIND, 96>(d, a, pdl, st);
        case 128: return chunk_launch<AT, KIND, 128>(d, a, pdl, st);
        case 192: return chunk_launch<AT, KIND, 192>(d, a, pdl, st);
        case 256: return chunk_launch<AT, KIND, 256>(d, a, pdl, st);
        default: return fail(JGPT_ERR_UNSUPPORTED, "key size %d", a.DK);
    }
}

int32_t launch_recurrent_chunks(bool f32, const StepDesc &d, const RecArgs &a, int pdl, cudaStream_t st) {
    if (d.n_chunks == 0) return JGPT_OK;
    switch (a.kind) {
        case REC_GLA: return f32 ? chunk_dispatch<float, REC_GLA>(d, a, pdl, st) : chunk_dispatch<__nv_bfloat16, REC_GLA>(d, a, pdl, st);
        case REC_DELTA: return f32 ? chunk_dispatch<float, REC_DELTA>(d, a, pdl, st) : chunk_dispatch<__nv_bfloat16, REC_DELTA>(d, a, pdl, st);
        case REC_HGRN2: return f32 ? chunk_dispatch<float, REC_HGRN2>(d, a, pdl, st) : chunk_dispatch<__nv_bfloat16, REC_HGRN2>(d, a, pdl, st);
        case REC_WKV: return f32 ? chunk_dispatch<float, REC_WKV>(d, a, pdl, st) : chunk_dispatch<__nv_bfloat16, REC_WKV>(d, a, pdl, st);
        case REC_GENERAL: return f32 ? chunk_dispatch<float, REC_GENERAL>(d, a, pdl, st) : chunk_dispatch<__nv_bfloat16, REC_GENERAL>(d, a, pdl, st);
    }
    return fail(JGPT_ERR_INVALID_ARGUMENT, "recurrence %d", a.kind);
}

}  // namespace mix
}  // namespace jgpt
