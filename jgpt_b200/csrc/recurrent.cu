// Recurrent mixers of the layered decoder, token by token: gated linear attention, the gated delta rule, the generalised delta rule, HGRN2 and WKV, all with
// a decay per key channel (long entries of a bf16 step take the chunked form, recurrent_chunk.cu), as ONE kernel from the layer's projections to the gated, normalised head outputs - for prompts, portions of
// prompts and single tokens alike, so a token's arithmetic does not depend on how its sequence was cut.
//
//   GLA    S <- diag(a) S + k v^T;                       o = S^T q
//   DELTA  S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q   (o read off as S_decayed^T q + (q.k) u)
//   GENERAL S <- diag(w) S - (a u) (u^T S) + k v^T with the old S on the right, u = k / n, n = |k|;  o = S^T q.  With s = S^T u:
//          S <- diag(w) S + u (n v)^T - (a u) s^T,  o read off as S^T (w q) - (q.(a u)) s + (q.u) n v
//   HGRN2  S <- diag(f) S + (1 - f) v^T;                 o = S^T q
//   WKV    o = (S + diag(u) k v^T)^T r, read off as S^T r + (r.(u k)) v;  S <- diag(w) S + k v^T
//
// A CTA owns one (sequence, head); a warp owns 16 value columns with every key row of the state in registers: lane =
// (row lane 0..7, column lane 0..3), DK / 8 rows x 4 columns, rows in pairs for the packed fp32 instructions
// (fma.rn.f32x2).  Tokens go through in tiles: the CTA first prepares a tile in shared memory (short convolution + silu,
// unit vectors, decays, step sizes), then every warp walks the tile's tokens on its own - no barrier inside - and the
// head outputs are normalised and gated from shared memory.  State and all of this arithmetic are fp32.
//
// State of a sequence and layer: S as [head][16-column group][DK][16] floats, then the convolution history
// [2][taps - 1][channels] of projection outputs.  The history has two copies: a step reads the one its entry names and
// writes the other, because heads that share query / key channels run in different CTAs.  Nothing is cleared when a slot
// is handed out: a step that starts at position 0 starts from zeros.
#include "recurrent_math.cuh"

#include <algorithm>
#include <type_traits>

namespace jgpt {
namespace mix {

// Tokens of a tile; fewer where two stages of raw rows would not fit.
__host__ __device__ constexpr int rec_tile_tokens(int kind, int DK, size_t elem) { return kind == REC_GENERAL && DK * elem > 192 * 4 ? 8 : 16; }

typedef unsigned long long u64;
__device__ __forceinline__ u64 pack2(float lo, float hi) {
    u64 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 unpack2(u64 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ u64 fma2(u64 a, u64 b, u64 c) {
    u64 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ u64 mul2(u64 a, u64 b) {
    u64 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// Eight sums over the eight row lanes (lane bits 2-4): on return a lane holds the total of value 4 * bit4 + 2 * bit3 + bit2.
__device__ __forceinline__ float reduce8(const float (&lo)[4], const float (&hi)[4], int lane) {
    const bool b4 = lane & 16, b3 = lane & 8, b2 = lane & 4;
    float r[4];
#pragma unroll
    for (int c = 0; c < 4; c++) r[c] = (b4 ? hi[c] : lo[c]) + __shfl_xor_sync(0xffffffffu, b4 ? lo[c] : hi[c], 16);
    float s[2];
#pragma unroll
    for (int c = 0; c < 2; c++) s[c] = (b3 ? r[c + 2] : r[c]) + __shfl_xor_sync(0xffffffffu, b3 ? r[c] : r[c + 2], 8);
    return (b2 ? s[1] : s[0]) + __shfl_xor_sync(0xffffffffu, b2 ? s[0] : s[1], 4);
}

// SINGLE: every listed entry has one token (a decode step): no tile loop, no staging ahead, CTAs of at most 256 threads kept
// small enough for several to share an SM, so that one's state is on its way while another computes.
__host__ __device__ constexpr int rec_single_blocks(int DK) { return DK <= 64 ? 3 : (DK <= 128 ? 2 : 1); }
template <class AT, int KIND, int DK, bool SINGLE>
__global__ void __launch_bounds__(SINGLE || DK > 128 ? 256 : 512, SINGLE ? rec_single_blocks(DK) : 1) recurrent_kernel(const RecArgs a, const Seg *__restrict__ segs, const int *__restrict__ list,
                                                                          int col_split, int tt,
                                                                          int pdl) {
    constexpr int NI = DK / 32;  // groups of four rows per lane
    extern __shared__ __align__(16) float rec_smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rl = lane >> 2, cl = lane & 3;
    const int nthreads = blockDim.x, nw = nthreads >> 5, DVc = nw * 16;
    const int h = blockIdx.x % a.heads, split = blockIdx.x / a.heads, col0 = split * DVc;
    constexpr int E = 16 / sizeof(AT);  // elements of a 16-byte chunk
    // a token's raw row: q, k, v, decay logits, output gate, then (delta) the chunk that holds its step size
    const int RK = DK, RV = rec_has_key(KIND) ? 2 * DK : DK, RZ = RV + DVc, RG = RZ + DK, RB = rec_has_gate(KIND) ? RG + DVc : RG,
              RW = RB + (KIND == REC_DELTA ? E : KIND == REC_GENERAL ? DK : 0);  // general: the removal rates' projection
    float *sq = rec_smem, *sk = sq + tt * DK, *sg = sk + tt * DK, *sa = sg + (rec_key_vectors(KIND) - 3) * tt * DK, *sv = sa + tt * DK, *so = sv + tt * DVc,
          *sbeta = so + tt * DVc, *sqk = sbeta + tt, *sqa = sqk + tt;
    AT *raw_s = reinterpret_cast<AT *>(sqk + (KIND == REC_GENERAL ? 3 : 1) * tt);  // [2][tt][RW]; one stage is enough for a single token

    if (pdl & 2) griddep_launch_dependents();
    const Seg sgm = segs[list[blockIdx.y]];
    if (sgm.seq < 0 || sgm.seq >= a.max_seqs) {
        if (tid == 0) atomicOr(a.status, DEV_STATUS_BAD_SEQ);
        return;
    }
    uint8_t *part = a.state + (uint64_t)sgm.seq * a.state_stride;
    float *S = reinterpret_cast<float *>(part) + ((size_t)h * (a.DV / 16) + col0 / 16 + warp) * (DK * 16);
    // no kernel of this step but this one touches this layer's state, and earlier steps are complete: read before the wait
    u64 st[NI * 2][4];
#pragma unroll
    for (int i = 0; i < NI * 2; i++) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
        if (sgm.pos0 > 0) {
            const float *row = S + (size_t)((i >> 1) * 32 + rl * 4 + (i & 1) * 2) * 16 + cl * 4;
            x = *reinterpret_cast<const float4 *>(row), y = *reinterpret_cast<const float4 *>(row + 16);
        }
        st[i][0] = pack2(x.x, y.x), st[i][1] = pack2(x.y, y.y), st[i][2] = pack2(x.z, y.z), st[i][3] = pack2(x.w, y.w);
    }
    if (pdl & 1) griddep_wait();

    const AT *__restrict__ proj = reinterpret_cast<const AT *>(a.proj) + (size_t)sgm.row0 * a.ldp;
    const AT *__restrict__ z = reinterpret_cast<const AT *>(a.z) + (size_t)sgm.row0 * a.ldz;
    const int kvh = h / (a.heads / a.kv_heads);
    const int nq = a.kv_heads * DK, channels = 2 * nq + a.heads * a.DV;  // convolution channels: q, k, v
    const AT *hist = reinterpret_cast<const AT *>(part + a.conv_off) + (size_t)sgm.conv_set * (a.taps > 0 ? a.taps - 1 : 0) * channels;
    const float qscale = rsqrtf((float)a.dim);
    const float rate = KIND == REC_DELTA ? expf(a.a_log[h]) : 1.f / a.tau;
    // the input of the convolution at token t of this entry (t < 0: history; before position 0: zero)
    auto conv_input = [&](int t, int proj_col, int channel) -> float2 {
        if (t >= 0) return load2(proj + (size_t)t * a.ldp + proj_col);
        if (sgm.pos0 + t >= 0) return load2(hist + (size_t)(-1 - t) * channels + channel);
        return make_float2(0.f, 0.f);
    };
    // channel pair idx of this CTA (q, then k, then its value columns): column in proj, convolution channel
    auto locate = [&](int idx, int &proj_col, int &channel) {
        if (idx < DK) {
            const bool is_k = idx >= DK / 2;
            const int c = kvh * DK + 2 * idx - (is_k ? DK : 0);
            proj_col = (is_k ? a.k_off : a.q_off) + c, channel = (is_k ? nq : 0) + c;
        } else {
            const int c = h * a.DV + col0 + 2 * (idx - DK);
            proj_col = a.v_off + c, channel = 2 * nq + c;
        }
    };
    const int npairs = DK + DVc / 2;
    // raw rows of a tile into stage `buf`
    auto stage = [&](int buf, int t0) {
        const int tn = SINGLE ? 1 : min(tt, sgm.T - t0), per = RW / E;
        for (int e = tid; e < tn * per; e += nthreads) {
            const int t = e / per, c = (e % per) * E;
            const AT *row = proj + (size_t)(t0 + t) * a.ldp, *zr = z + (size_t)(t0 + t) * a.ldz, *src;
            if (c < RK) src = row + a.q_off + kvh * DK + c;
            else if (c < RV) src = row + a.k_off + kvh * DK + c - RK;
            else if (c < RZ) src = row + a.v_off + h * a.DV + col0 + c - RV;
            else if (c < RG) src = zr + a.z_off + h * DK + c - RZ;
            else if (c < RB) src = (KIND == REC_DELTA ? zr + a.zg_off : row + a.g_off) + h * a.DV + col0 + c - RG;
            else src = KIND == REC_GENERAL ? row + a.b_off + h * DK + c - RB : row + a.b_off + h / E * E;
            cp_async16(raw_s + ((size_t)buf * tt + t) * RW + c, src, true);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // convolution + silu of one channel pair over the tile
    auto convolve = [&](auto max_taps, int idx, const AT *raw, const AT *prev, int t0, int tn, float *dst, int ld) {
        constexpr int MT = decltype(max_taps)::value;
        int pc, ch;
        locate(idx, pc, ch);
        const float *w = (ch < nq ? a.conv_q + (size_t)ch * a.taps
                                  : (ch < 2 * nq ? a.conv_k + (size_t)(ch - nq) * a.taps : a.conv_v + (size_t)(ch - 2 * nq) * a.taps));
        float2 wt[MT], win[MT];  // right-aligned: entry MT - 1 is the current token's
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const int back = MT - 1 - i;
            const bool on = back < a.taps;
            wt[i] = on ? make_float2(w[a.taps - 1 - back], w[2 * a.taps - 1 - back]) : make_float2(0.f, 0.f);
            // the window in front of the tile's first token: entry i holds token t0 - back
            win[i] = !on || back == 0 ? make_float2(0.f, 0.f) : (t0 > 0 ? load2(prev + (size_t)(tt - back) * RW + 2 * idx) : conv_input(-back, pc, ch));
        }
#pragma unroll 4
        for (int t = 0; t < tn; t++) {
            win[MT - 1] = load2(raw + (size_t)t * RW + 2 * idx);
            float2 y = make_float2(0.f, 0.f);
#pragma unroll
            for (int i = 0; i < MT; i++) y.x = fmaf(wt[i].x, win[i].x, y.x), y.y = fmaf(wt[i].y, win[i].y, y.y);
            y.x *= sigmoid_f<AT>(y.x), y.y *= sigmoid_f<AT>(y.y);
            *reinterpret_cast<float2 *>(dst + t * ld) = y;
#pragma unroll
            for (int i = 0; i + 1 < MT; i++) win[i] = win[i + 1];
        }
    };
    stage(0, 0);
    for (int t0 = 0, buf = 0; t0 < (SINGLE ? 1 : sgm.T); t0 += tt, buf ^= 1) {
        const int tn = SINGLE ? 1 : min(tt, sgm.T - t0);
        const AT *raw = raw_s + (size_t)buf * tt * RW, *prev = raw_s + (size_t)(buf ^ 1) * tt * RW;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        // ---- prepare the tile ----
        for (int idx = tid; idx < npairs; idx += nthreads) {
            float *dst = idx < DK / 2 ? sq + 2 * idx : (idx < DK ? sk + 2 * idx - DK : sv + 2 * (idx - DK));
            const int ld = idx < DK ? DK : DVc;
            if (KIND == REC_DELTA) {
                if (a.taps <= 4) convolve(std::integral_constant<int, 4>(), idx, raw, prev, t0, tn, dst, ld);
                else convolve(std::integral_constant<int, kMaxTaps>(), idx, raw, prev, t0, tn, dst, ld);
            } else {
                if (!rec_has_key(KIND) && idx >= DK / 2 && idx < DK) {  // its key comes with the forget gate
                    if (!SINGLE && (tn & 1)) *reinterpret_cast<float2 *>(dst + tn * ld) = make_float2(0.f, 0.f);
                    continue;
                }
                const float f = KIND == REC_GLA && idx < DK / 2 ? qscale : 1.f;
                const int from = idx < DK ? 2 * idx : RV + 2 * (idx - DK);
#pragma unroll 4
                for (int t = 0; t < tn; t++) {
                    float2 y = load2(raw + (size_t)t * RW + from);
                    if (KIND == REC_HGRN2 && idx < DK / 2) y.x *= sigmoid_f<AT>(y.x), y.y *= sigmoid_f<AT>(y.y);
                    else y.x *= f, y.y *= f;
                    *reinterpret_cast<float2 *>(dst + t * ld) = y;
                }
                if (!SINGLE && (tn & 1)) *reinterpret_cast<float2 *>(dst + tn * ld) = make_float2(0.f, 0.f);  // pads the last pair of tokens
            }
        }
        for (int idx = tid; idx < tn * (DK / 2); idx += nthreads) {
            const int t = idx / (DK / 2), c = 2 * (idx % (DK / 2));
            float2 y = load2(raw + (size_t)t * RW + RZ + c);
            const float2 b = *reinterpret_cast<const float2 *>(a.decay_bias + h * DK + c);
            y.x += b.x, y.y += b.y;
            if (KIND == REC_GLA) y.x = -y.x, y.y = -y.y;  // sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
            if (KIND == REC_HGRN2) {
                const float2 low = *reinterpret_cast<const float2 *>(a.lower + h * DK + c);
                const float2 f0 = forget_write<AT>(y.x, low.x), f1 = forget_write<AT>(y.y, low.y);
                y = make_float2(f0.x, f1.x);
                *reinterpret_cast<float2 *>(sk + t * DK + c) = make_float2(f0.y, f1.y);
            } else if (KIND == REC_WKV) {
                y.x = exp_neg_exp<AT>(y.x), y.y = exp_neg_exp<AT>(y.y);
            } else if (KIND == REC_GENERAL) {
                y.x = exp_f<AT>(-a.rate * sigmoid_f<AT>(y.x)), y.y = exp_f<AT>(-a.rate * sigmoid_f<AT>(y.y));
                float2 m = load2(raw + (size_t)t * RW + RB + c);
                const float2 mb = *reinterpret_cast<const float2 *>(a.removal_bias + h * DK + c);
                m.x = sigmoid_f<AT>(m.x + mb.x), m.y = sigmoid_f<AT>(m.y + mb.y);
                *reinterpret_cast<float2 *>(sa + t * DK + c) = m;
            } else {
                y.x = exp_f<AT>(-rate * softplus_f<AT>(y.x)), y.y = exp_f<AT>(-rate * softplus_f<AT>(y.y));
            }
            *reinterpret_cast<float2 *>(sg + t * DK + c) = y;
        }
        if (!SINGLE && KIND != REC_DELTA && KIND != REC_GENERAL && (tn & 1))
            for (int c = tid; c < DK; c += nthreads) sg[tn * DK + c] = 1.f;
        __syncthreads();
        if (!SINGLE && t0 + tt < sgm.T) stage(buf ^ 1, t0 + tt);  // lands while this tile runs; the previous tile's rows are no longer needed
        if (KIND == REC_DELTA) {
            for (int t = warp; t < tn; t += nw) {
                float qv[NI], kv[NI], qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
                for (int i = 0; i < NI; i++) {
                    qv[i] = sq[t * DK + lane + 32 * i], kv[i] = sk[t * DK + lane + 32 * i];
                    qq += qv[i] * qv[i], kk += kv[i] * kv[i], qk += qv[i] * kv[i];
                }
                qq = warp_sum(qq), kk = warp_sum(kk), qk = warp_sum(qk);
                const float fq = qscale / sqrtf(qq + 1e-6f), fk = 1.f / sqrtf(kk + 1e-6f);
#pragma unroll
                for (int i = 0; i < NI; i++) sq[t * DK + lane + 32 * i] = qv[i] * fq, sk[t * DK + lane + 32 * i] = kv[i] * fk;
                if (lane == 0) sqk[t] = qk * fq * fk, sbeta[t] = sigmoid_f<AT>(load1(raw + (size_t)t * RW + RB + h % E));
            }
            __syncthreads();
        }
        if (KIND == REC_GENERAL) {
            for (int t = warp; t < tn; t += nw) {
                float kv[NI], kk = 0.f, qu = 0.f, qa = 0.f;
#pragma unroll
                for (int i = 0; i < NI; i++) kv[i] = sk[t * DK + lane + 32 * i], kk += kv[i] * kv[i];
                const float n = sqrtf(warp_sum(kk) + 1e-6f), f = 1.f / n;
#pragma unroll
                for (int i = 0; i < NI; i++) {
                    const int at = t * DK + lane + 32 * i;
                    const float u = kv[i] * f, au = sa[at] * u, q = sq[at];
                    qu += q * u, qa += q * au;
                    sk[at] = u, sa[at] = au, sq[at] = q * sg[at];
                }
                qu = warp_sum(qu), qa = warp_sum(qa);
                if (lane == 0) sbeta[t] = n, sqk[t] = qu, sqa[t] = qa;
            }
            __syncthreads();
        }
        if (KIND == REC_WKV) {  // what the current token adds to its own output: (r . (u k)) v
            for (int t = warp; t < tn; t += nw) {
                float rk = 0.f;
#pragma unroll
                for (int i = 0; i < NI; i++) rk += sq[t * DK + lane + 32 * i] * sk[t * DK + lane + 32 * i] * a.bonus[h * DK + lane + 32 * i];
                rk = warp_sum(rk);
                if (lane == 0) sqk[t] = rk;
            }
            __syncthreads();
        }
        // ---- the recurrence: every warp on its own columns ----
        const int vcol = warp * 16 + cl * 4;
        if (KIND == REC_GENERAL) {
            for (int t = 0; t < tn; t++) {
                u64 ks[4] = {0, 0, 0, 0}, qs[4] = {0, 0, 0, 0};
                const float *qp = sq + t * DK + rl * 4, *kp = sk + t * DK + rl * 4, *gp = sg + t * DK + rl * 4, *ap = sa + t * DK + rl * 4;
#pragma unroll
                for (int i = 0; i < NI; i++) {
                    const ulonglong2 q2 = *reinterpret_cast<const ulonglong2 *>(qp + 32 * i), k2 = *reinterpret_cast<const ulonglong2 *>(kp + 32 * i);
#pragma unroll
                    for (int c = 0; c < 4; c++) {
                        ks[c] = fma2(k2.x, st[2 * i][c], ks[c]), ks[c] = fma2(k2.y, st[2 * i + 1][c], ks[c]);
                        qs[c] = fma2(q2.x, st[2 * i][c], qs[c]), qs[c] = fma2(q2.y, st[2 * i + 1][c], qs[c]);
                    }
                }
                float kf[4], qf[4];
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    const float2 x = unpack2(ks[c]), y = unpack2(qs[c]);
                    kf[c] = x.x + x.y, qf[c] = y.x + y.y;
                }
                const float tot = reduce8(kf, qf, lane);
                const float4 v4 = *reinterpret_cast<const float4 *>(sv + t * DVc + vcol);
                const float n = sbeta[t];
                float nv[4], s[4];
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    s[c] = __shfl_sync(0xffffffffu, tot, ((c & 2) << 2) | ((c & 1) << 2) | cl);
                    nv[c] = n * (c == 0 ? v4.x : c == 1 ? v4.y : c == 2 ? v4.z : v4.w);
                }
                if (lane & 16) {
                    const int c = rl & 3;
                    const float sc = c == 0 ? s[0] : c == 1 ? s[1] : c == 2 ? s[2] : s[3], nc = c == 0 ? nv[0] : c == 1 ? nv[1] : c == 2 ? nv[2] : nv[3];
                    so[t * DVc + vcol + c] = fmaf(sqk[t], nc, fmaf(-sqa[t], sc, tot));
                }
                u64 n2[4], s2[4];
#pragma unroll
                for (int c = 0; c < 4; c++) n2[c] = pack2(nv[c], nv[c]), s2[c] = pack2(-s[c], -s[c]);
#pragma unroll
                for (int i = 0; i < NI; i++) {
                    const ulonglong2 k2 = *reinterpret_cast<const ulonglong2 *>(kp + 32 * i), g2 = *reinterpret_cast<const ulonglong2 *>(gp + 32 * i),
                                     a2 = *reinterpret_cast<const ulonglong2 *>(ap + 32 * i);
#pragma unroll
                    for (int c = 0; c < 4; c++) {
                        st[2 * i][c] = fma2(a2.x, s2[c], fma2(k2.x, n2[c], mul2(g2.x, st[2 * i][c])));
                        st[2 * i + 1][c] = fma2(a2.y, s2[c], fma2(k2.y, n2[c], mul2(g2.y, st[2 * i + 1][c])));
                    }
                }
            }
        } else if (KIND == REC_DELTA) {
            for (int t = 0; t < tn; t++) {
                u64 ks[4] = {0, 0, 0, 0}, qs[4] = {0, 0, 0, 0};
                const float *qp = sq + t * DK + rl * 4, *kp = sk + t * DK + rl * 4, *gp = sg + t * DK + rl * 4;
#pragma unroll
                for (int i = 0; i < NI; i++) {
                    const ulonglong2 q2 = *reinterpret_cast<const ulonglong2 *>(qp + 32 * i);
                    const ulonglong2 k2 = *reinterpret_cast<const ulonglong2 *>(kp + 32 * i);
                    const ulonglong2 g2 = *reinterpret_cast<const ulonglong2 *>(gp + 32 * i);
#pragma unroll
                    for (int c = 0; c < 4; c++) {
                        st[2 * i][c] = mul2(g2.x, st[2 * i][c]);
                        st[2 * i + 1][c] = mul2(g2.y, st[2 * i + 1][c]);
                        ks[c] = fma2(k2.x, st[2 * i][c], ks[c]), ks[c] = fma2(k2.y, st[2 * i + 1][c], ks[c]);
                        qs[c] = fma2(q2.x, st[2 * i][c], qs[c]), qs[c] = fma2(q2.y, st[2 * i + 1][c], qs[c]);
                    }
                }
                float kf[4], qf[4];
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    const float2 x = unpack2(ks[c]), y = unpack2(qs[c]);
                    kf[c] = x.x + x.y, qf[c] = y.x + y.y;
                }
                const float tot = reduce8(kf, qf, lane);
                const float4 v4 = *reinterpret_cast<const float4 *>(sv + t * DVc + vcol);
                const float beta = sbeta[t];
                float u[4];
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    const float sk_c = __shfl_sync(0xffffffffu, tot, ((c & 2) << 2) | ((c & 1) << 2) | cl);
                    u[c] = beta * ((c == 0 ? v4.x : c == 1 ? v4.y : c == 2 ? v4.z : v4.w) - sk_c);
                }
                if (lane & 16) {
                    const int c = rl & 3;
                    const float uc = c == 0 ? u[0] : c == 1 ? u[1] : c == 2 ? u[2] : u[3];
                    so[t * DVc + vcol + c] = fmaf(sqk[t], uc, tot);
                }
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    const u64 u2 = pack2(u[c], u[c]);
#pragma unroll
                    for (int i = 0; i < NI; i++) {
                        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2 *>(kp + 32 * i);
                        st[2 * i][c] = fma2(k2.x, u2, st[2 * i][c]), st[2 * i + 1][c] = fma2(k2.y, u2, st[2 * i + 1][c]);
                    }
                }
            }
        } else {
            for (int t = 0; t < tn; t += 2) {
                float of[2][4] = {};
#pragma unroll
                for (int e = 0; e < (SINGLE ? 1 : 2); e++) {
                    u64 qs[4] = {0, 0, 0, 0}, v2[4];
                    const float *qp = sq + (t + e) * DK + rl * 4, *kp = sk + (t + e) * DK + rl * 4, *gp = sg + (t + e) * DK + rl * 4;
                    const float4 v4 = *reinterpret_cast<const float4 *>(sv + (t + e) * DVc + vcol);
                    v2[0] = pack2(v4.x, v4.x), v2[1] = pack2(v4.y, v4.y), v2[2] = pack2(v4.z, v4.z), v2[3] = pack2(v4.w, v4.w);
#pragma unroll
                    for (int i = 0; i < NI; i++) {
                        const ulonglong2 q2 = *reinterpret_cast<const ulonglong2 *>(qp + 32 * i);
                        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2 *>(kp + 32 * i);
                        const ulonglong2 g2 = *reinterpret_cast<const ulonglong2 *>(gp + 32 * i);
#pragma unroll
                        for (int c = 0; c < 4; c++) {
                            if (KIND == REC_WKV) qs[c] = fma2(q2.x, st[2 * i][c], qs[c]), qs[c] = fma2(q2.y, st[2 * i + 1][c], qs[c]);
                            st[2 * i][c] = fma2(k2.x, v2[c], mul2(g2.x, st[2 * i][c]));
                            st[2 * i + 1][c] = fma2(k2.y, v2[c], mul2(g2.y, st[2 * i + 1][c]));
                            if (KIND != REC_WKV) qs[c] = fma2(q2.x, st[2 * i][c], qs[c]), qs[c] = fma2(q2.y, st[2 * i + 1][c], qs[c]);
                        }
                    }
#pragma unroll
                    for (int c = 0; c < 4; c++) {
                        const float2 y = unpack2(qs[c]);
                        of[e][c] = y.x + y.y;
                    }
                }
                float tot = reduce8(of[0], of[1], lane);
                if (KIND == REC_WKV && t + (lane >> 4) < tn) tot = fmaf(sqk[t + (lane >> 4)], sv[(t + (lane >> 4)) * DVc + vcol + (rl & 3)], tot);
                if (!SINGLE || lane < 16) so[(t + (lane >> 4)) * DVc + vcol + (rl & 3)] = tot;  // row tn of an odd tile is a spare
            }
        }
        __syncthreads();
        // ---- head outputs: RMS norm over the value columns, gate ----
        if (col_split > 1) {
            for (int idx = tid; idx < tn * DVc; idx += nthreads)
                a.raw[(size_t)(sgm.row0 + t0 + idx / DVc) * (a.heads * a.DV) + h * a.DV + col0 + idx % DVc] = so[idx];
        } else {
            for (int t = warp; t < tn; t += nw) {
                float ss = 0.f;
                for (int c = lane; c < DVc; c += 32) {
                    const float v = so[t * DVc + c];
                    ss += v * v;
                }
                const float inv = a.out_scale / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
                AT *o = reinterpret_cast<AT *>(a.out) + (size_t)(sgm.row0 + t0 + t) * a.ldo + a.out_off + h * DVc;
                const AT *gp = raw + (size_t)t * RW + RG;
                const float *nm = a.norm_w + h * a.norm_stride;
                for (int c = lane; c < DVc; c += 32)
                    store1(o + c, so[t * DVc + c] * inv * nm[c] * (rec_has_gate(KIND) ? out_gate<AT, KIND>(load1(gp + c)) : 1.f));
            }
        }
    }
    // ---- leave the state for the next step ----
#pragma unroll
    for (int i = 0; i < NI * 2; i++) {
        float *row = S + (size_t)((i >> 1) * 32 + rl * 4 + (i & 1) * 2) * 16 + cl * 4;
        const float2 c0 = unpack2(st[i][0]), c1 = unpack2(st[i][1]), c2 = unpack2(st[i][2]), c3 = unpack2(st[i][3]);
        *reinterpret_cast<float4 *>(row) = make_float4(c0.x, c1.x, c2.x, c3.x);
        *reinterpret_cast<float4 *>(row + 16) = make_float4(c0.y, c1.y, c2.y, c3.y);
    }
    if (KIND == REC_DELTA && a.taps > 1) {
        AT *next = reinterpret_cast<AT *>(part + a.conv_off) + (size_t)(1 - sgm.conv_set) * (a.taps - 1) * channels;
        const bool first_of_group = h % (a.heads / a.kv_heads) == 0 && split == 0;
        for (int idx = tid; idx < npairs; idx += nthreads) {
            if (idx < DK && !first_of_group) continue;  // shared channels are written once
            int pc, ch;
            locate(idx, pc, ch);
            for (int i = 0; i < a.taps - 1; i++) store2(next + (size_t)i * channels + ch, conv_input(sgm.T - 1 - i, pc, ch));
        }
    }
}

// RMS norm and gate of heads whose columns were cut over several CTAs.
template <class AT, int KIND>
__global__ void __launch_bounds__(256) gated_norm_kernel(const RecArgs a, int rows) {
    const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    const int per = norm_heads_per_warp(a.DV), groups = (a.heads + per - 1) / per;
    if (item >= rows * groups) return;
    norm_gate_group<AT, KIND>(a, item / groups, item % groups * per, lane);
}

int rec_padded_key(int dim) {
    for (int d : {32, 64, 96, 128, 192, 256})
        if (dim <= d) return dim > 0 ? d : 0;
    return 0;
}
int rec_padded_value(int vdim) { return vdim > 0 && vdim <= 256 ? (vdim + 15) / 16 * 16 : 0; }

uint64_t rec_state_bytes(const RecArgs &a, int elem_bytes, uint64_t *conv_off) {
    const uint64_t s = (uint64_t)a.heads * a.DK * a.DV * sizeof(float);
    *conv_off = s;  // the convolution's history, or WKV's previous rows
    const uint64_t channels = 2ull * a.kv_heads * a.DK + (uint64_t)a.heads * a.DV;
    const uint64_t conv = a.taps > 1 ? 2ull * (uint64_t)(a.taps - 1) * channels * (uint64_t)elem_bytes : 0;
    return (s + conv + 2 * sizeof(float) * (uint64_t)a.shift_width + 255) / 256 * 256;
}

template <class AT, int KIND, int DK, bool SINGLE>
static int32_t rec_launch_form(const StepDesc &d, const RecArgs &a, int pdl, int *split_out, cudaStream_t st) {
    const bool single = SINGLE;
    constexpr int tile_tokens = rec_tile_tokens(KIND, DK, sizeof(AT));
    const int tt = single ? 2 : tile_tokens;
    const int groups = a.DV / 16, max_groups = DK <= 128 && !SINGLE ? 16 : 8;
    int split = 1;
    auto allowed = [&](int s) { return groups % s == 0; };
    while (split < groups && (!allowed(split) || groups / split > max_groups)) split++;
    *split_out = split;
    const int nw = groups / split, DVc = nw * 16;
    auto smem_bytes = [](int tokens, int cols, int stages) {
        const size_t row = rec_key_vectors(KIND) * DK + 2 * (size_t)cols;
        return sizeof(float) * ((size_t)tokens * row + (KIND == REC_GENERAL ? 4 : 2) * tokens) + (size_t)stages * tokens * (row * sizeof(AT) + (KIND == REC_DELTA ? 16 : 0));
    };
    const size_t smem = smem_bytes(tt, DVc, single ? 1 : 2);
    auto kern = recurrent_kernel<AT, KIND, DK, SINGLE>;
    static thread_local int set_for = -1;
    int dev = 0;
    JGPT_CUDA_TRY(cudaGetDevice(&dev));
    if (set_for != dev) {
        JGPT_CUDA_TRY(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_bytes(tile_tokens, 16 * max_groups, 2)));
        set_for = dev;
    }
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = dim3((unsigned)(a.heads * split), (unsigned)d.n_short), cfg.blockDim = dim3((unsigned)(32 * nw));
    cfg.dynamicSmemBytes = smem, cfg.stream = st, cfg.attrs = attr, cfg.numAttrs = (pdl & 1) ? 1 : 0;
    JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, kern, a, d.segs, d.short_segs, split, tt, pdl));
    return JGPT_OK;
}

template <class AT, int KIND, int DK>
static int32_t rec_launch(const StepDesc &d, const RecArgs &a, int pdl, int *split_out, cudaStream_t st) {
    if (d.n_short == 0) return JGPT_OK;
    // heads wider than a single-token CTA's 128 columns keep the tile form, which normalises them without a second kernel
    if (d.n_tiles == 0 && (a.DV <= 128 || DK > 128)) return rec_launch_form<AT, KIND, DK, true>(d, a, pdl, split_out, st);
    return rec_launch_form<AT, KIND, DK, false>(d, a, pdl, split_out, st);
}

template <class AT, int KIND>
static int32_t rec_run(const StepDesc &d, const RecArgs &a, int pdl, cudaStream_t st) {
    int split = 1;
    int32_t rc = launch_recurrent_chunks(sizeof(AT) == 4, d, a, pdl, st);
    if (!rc)
        switch (a.DK) {
            case 32: rc = rec_launch<AT, KIND, 32>(d, a, pdl, &split, st); break;
            case 64: rc = rec_launch<AT, KIND, 64>(d, a, pdl, &split, st); break;
            case 96: rc = rec_launch<AT, KIND, 96>(d, a, pdl, &split, st); break;
            case 128: rc = rec_launch<AT, KIND, 128>(d, a, pdl, &split, st); break;
            case 192: rc = rec_launch<AT, KIND, 192>(d, a, pdl, &split, st); break;
            case 256: rc = rec_launch<AT, KIND, 256>(d, a, pdl, &split, st); break;
            default: return fail(JGPT_ERR_UNSUPPORTED, "key size %d", a.DK);
        }
    if (rc) return rc;
    if (split > 1) {  // raw outputs of every row: the chunked rows are normed here as well (once more, to the same values)
        gated_norm_kernel<AT, KIND><<<(unsigned)((d.rows * a.heads + 7) / 8), 256, 0, st>>>(a, d.rows);
        JGPT_CUDA_TRY(cudaGetLastError());
    }
    return JGPT_OK;
}

int32_t launch_recurrent(bool f32, const StepDesc &d, const RecArgs &a, int pdl, cudaStream_t st) {
    JGPT_REQUIRE(a.taps <= kMaxTaps, JGPT_ERR_UNSUPPORTED, "convolutions of up to %d taps", kMaxTaps);
    switch (a.kind) {
        case REC_GLA: return f32 ? rec_run<float, REC_GLA>(d, a, pdl, st) : rec_run<__nv_bfloat16, REC_GLA>(d, a, pdl, st);
        case REC_DELTA: return f32 ? rec_run<float, REC_DELTA>(d, a, pdl, st) : rec_run<__nv_bfloat16, REC_DELTA>(d, a, pdl, st);
        case REC_HGRN2: return f32 ? rec_run<float, REC_HGRN2>(d, a, pdl, st) : rec_run<__nv_bfloat16, REC_HGRN2>(d, a, pdl, st);
        case REC_WKV: return f32 ? rec_run<float, REC_WKV>(d, a, pdl, st) : rec_run<__nv_bfloat16, REC_WKV>(d, a, pdl, st);
        case REC_GENERAL: return f32 ? rec_run<float, REC_GENERAL>(d, a, pdl, st) : rec_run<__nv_bfloat16, REC_GENERAL>(d, a, pdl, st);
    }
    return fail(JGPT_ERR_INVALID_ARGUMENT, "recurrence %d", a.kind);
}

}  // namespace mix
}  // namespace jgpt
