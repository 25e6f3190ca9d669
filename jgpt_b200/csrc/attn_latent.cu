// Latent attention of the layered decoder: a page row holds the normed latent c and one rotated key part shared by all heads,
// and a query sees a sliding window (or everything before it).
//
//   latent_prep_kernel    norms of the query and key latents, rotation of the key part, append to the pages
//   latent_rows_kernel    one warp per (row, head), fp32: the exact mode
//   latent_attn_kernel    bf16 on the latents themselves (scores q~ . c + q_rot . k_rot with q~ = W_uk^T q, values c): single
//                         tokens over a cluster-split window, short portions of prompts
//   latent_gather_kernel, latent_tile_kernel
//                         long portions: keys and values of the visible positions written out per head in a workspace (a plain
//                         product of the gathered latents), then tiles of query tokens against tiles of keys
//
// On the latents every head reads the same 64 staged rows, so a decoded token costs one trip through its window; written out a
// (query, key) pair costs dim + rot_dim + vdim multiply-adds per head instead of 2 kv_rank + rot_dim.
#include "attn_mma.cuh"

#include <algorithm>

namespace jgpt {
namespace mix {

__host__ __device__ __forceinline__ int window_first(int pos, int window) { return window > 0 && pos >= window ? pos - window + 1 : 0; }

// Element j of a rotated vector at `x` (its first 2 half dimensions turn, the rest pass), cs = this row's angles.
template <class AT>
__device__ __forceinline__ float rotated(const AT *x, const float2 *cs, int half, int j) {
    if (j >= 2 * half) return act_load(x + j);
    const int i = j < half ? j : j - half;
    const float u = act_load(x + i), v = act_load(x + half + i);
    const float2 t = cs[i];
    return j < half ? u * t.x - v * t.y : v * t.x + u * t.y;
}

// A warp per (row, part): part 0 the query latent, part 1 the key latent and the rotated part.  Latents start at multiples of
// eight columns and are followed by zeros up to the next one.
template <class AT>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int rows, int pdl) {
    constexpr int NV = 4;  // the first 1024 elements stay in registers
    const int item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31, parts = a.own_cache ? 2 : 1;
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    if (item >= rows * parts) return;
    const int r = item / parts, part = item % parts;
    const AT *proj = reinterpret_cast<const AT *>(a.proj) + (size_t)r * a.ldp;
    const AT *src = proj + (part ? a.c_off : a.dq_off);
    const float *gamma = part ? a.dkv_norm : a.dq_norm;
    const int n = part ? a.kv_rank : a.q_rank, padded = part ? a.KR : a.ldcq;
    AT *dst = reinterpret_cast<AT *>(a.cq) + (size_t)r * a.ldcq;
    if (part) {
        const int phys = page_of(a, seq[r], pos[r]);
        if (phys < 0) return;
        dst = reinterpret_cast<AT *>(a.kv) + ((size_t)phys * kBlockTokens + pos[r] % kBlockTokens) * a.LDR;
    }
    float v[NV][8], ss = 0.f;
    auto squares = [&](const float (&x)[8]) {
#pragma unroll
        for (int e = 0; e < 8; e++) ss += x[e] * x[e];
    };
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int j = (lane + 32 * i) * 8;
        if (j < n) load8(src + j, v[i]);
        else {
#pragma unroll
            for (int e = 0; e < 8; e++) v[i][e] = 0.f;
        }
        squares(v[i]);
    }
    for (int j = (lane + 32 * NV) * 8; j < n; j += 256) {
        float x[8];
        load8(src + j, x), squares(x);
    }
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    const float inv = 1.f / sqrtf(ss / (float)n + a.eps);
    auto put = [&](int j, float (&x)[8]) {
#pragma unroll
        for (int e = 0; e < 8; e++) x[e] = j + e < n ? x[e] * inv * __ldg(gamma + j + e) : 0.f;
        store8(dst + j, x);
    };
#pragma unroll
    for (int i = 0; i < NV; i++)
        if ((lane + 32 * i) * 8 < padded) put((lane + 32 * i) * 8, v[i]);
    for (int j = (lane + 32 * NV) * 8; j < padded; j += 256) {
        float x[8];
        load8(src + min(j, (n - 1) / 8 * 8), x), put(j, x);
    }
    if (part)
        for (int j = lane; j < a.RR; j += 32)
            act_store(dst + a.KR + j, j < a.rot_dim ? rotated(proj + a.r_off, a.cs + (size_t)r * a.half, a.half, j) : 0.f);
}

constexpr int kMaxRank = 512, kMaxRot = 128;

// One warp per (row, head): lane l holds elements l, l + 32, ... of q~, of the rotated part and of the weighted sum.
template <class AT>
__global__ void __launch_bounds__(256) latent_rows_kernel(const LatentArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int rows) {
    constexpr int NC = kMaxRank / 32, NR = kMaxRot / 32;
    const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= rows * a.heads) return;
    const int r = item / a.heads, h = item % a.heads, nc = a.KR / 32;
    AT *qa = reinterpret_cast<AT *>(a.qa) + (size_t)r * a.heads * a.KR + (size_t)h * a.KR + lane;
    const AT *qr = reinterpret_cast<const AT *>(a.q) + (size_t)r * a.ldq + (size_t)h * a.DQ + a.DP;
    float q[NC], o[NC], qrot[NR];
#pragma unroll
    for (int e = 0; e < NC; e++) q[e] = e < nc ? act_load(qa + 32 * e) * a.scale : 0.f, o[e] = 0.f;
#pragma unroll
    for (int e = 0; e < NR; e++)
        qrot[e] = lane + 32 * e < a.rot_dim ? rotated(qr, a.cs + (size_t)r * a.half, a.half, lane + 32 * e) * a.scale : 0.f;
    float m = -INFINITY, l = 0.f;
    const int p = pos[r], s = seq[r];
    for (int j = window_first(p, a.window); j <= p; j++) {
        const int phys = page_of(a, s, j);
        if (phys < 0) break;
        const AT *row = reinterpret_cast<const AT *>(a.kv) + ((size_t)phys * kBlockTokens + j % kBlockTokens) * a.LDR + lane;
        float c[NC], d = 0.f;
#pragma unroll
        for (int e = 0; e < NC; e++) {
            c[e] = e < nc ? act_load(row + 32 * e) : 0.f;
            d = fmaf(q[e], c[e], d);
        }
#pragma unroll
        for (int e = 0; e < NR; e++)
            if (lane + 32 * e < a.rot_dim) d = fmaf(qrot[e], act_load(row + a.KR + 32 * e), d);
#pragma unroll
        for (int off = 16; off >= 1; off >>= 1) d += __shfl_xor_sync(0xffffffffu, d, off);
        const float mn = fmaxf(m, d), f = expf(m - mn), w = expf(d - mn);
        m = mn, l = l * f + w;
#pragma unroll
        for (int e = 0; e < NC; e++) o[e] = fmaf(w, c[e], o[e] * f);
    }
    const float f = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
    for (int e = 0; e < NC; e++)
        if (e < nc) act_store(qa + 32 * e, o[e] * f);
}

// ------------------------------------------------------------------------------------------------
// On the latents, bf16
// ------------------------------------------------------------------------------------------------
// CTA = 16 MT (token, head) rows of an entry, eight warps and a ninth that brings in tiles of 32 keys = two pages by bulk copies (a
// page is contiguous, its row stride an odd number of 16-byte units, so ldmatrix is free of bank conflicts).  A warp scores the
// tile's keys over an eighth of the row's elements (its part of the query rows stays in registers: shared memory bandwidth is what
// a tile costs); the parts meet in shared memory, where every warp turns an eighth of the rows into weights (bf16 high and low
// parts) and then adds up its eighth of the latent's columns.  A cluster splits the keys; partial sums
// meet through cluster shared memory.
constexpr int kLatKeys = 32, kLatPages = kLatKeys / kBlockTokens, kLatLS = kLatKeys + 8, kLatThreads = 288;
constexpr size_t kMaxSmem = 232448 - 4096;  // dynamic; the rest is for static shared memory

template <int MT>
__host__ __device__ constexpr size_t latent_fixed_smem(int LDR) {
    const size_t query = (size_t)16 * MT * LDR * 2, scores = sizeof(float) * 8 * 16 * MT * kLatLS;  // one after the other in the same place
    return (query > scores ? query : scores) + 2 * (size_t)16 * MT * kLatLS * 2;
}

template <int NTW, int MT>
__global__ void __launch_bounds__(kLatThreads, MT == 1 ? 2 : 1) latent_attn_kernel(const LatentArgs a, const Seg *__restrict__ segs, int stages, int pdl) {
    constexpr int KR = NTW * 64, ROWS = 16 * MT, MAXST = 8, TPR = 256 / ROWS;
    extern __shared__ __align__(128) uint8_t lat_smem[];
    __shared__ __align__(8) uint64_t full[MAXST], empty[MAXST];
    __shared__ int s_abort_mem;
    __shared__ float s_ml[8][ROWS][2];           // row maxima and sums of every CTA of the cluster
    __shared__ float s_m[ROWS], s_l[ROWS], s_f[ROWS];  // this CTA's running maxima, sums, the last tile's factors
    volatile int *s_abort = &s_abort_mem;
    const int LDR = a.LDR, RR = a.RR, H = a.heads;
    const uint32_t page_bytes = (uint32_t)(kBlockTokens * LDR * 2);
    __nv_bfloat16 *ring = reinterpret_cast<__nv_bfloat16 *>(lat_smem);     // [stages][32][LDR]
    __nv_bfloat16 *ph = ring + (size_t)stages * kLatKeys * LDR, *pl = ph + ROWS * kLatLS;  // [ROWS][kLatLS] weights
    __nv_bfloat16 *qs = pl + ROWS * kLatLS;                                // [ROWS][LDR], until the operands are in registers
    float *sp = reinterpret_cast<float *>(qs);                             // [8][ROWS][kLatLS] parts of the scores
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = 2 * (lane & 3);
    const int nsplit = gridDim.x, split = blockIdx.x, r0 = blockIdx.y * ROWS;
    if (pdl & 2) griddep_launch_dependents();
    const Seg sg = segs[blockIdx.z];
    const int rows = sg.T * H;
    if (r0 >= rows) return;  // the whole cluster
    if (nsplit > 1) cluster_arrive();
    const int first = window_first(sg.pos0 + r0 / H, a.window), last = sg.pos0 + min(rows - 1, r0 + ROWS - 1) / H;
    const int lo_page = first / kBlockTokens, n_pages = last / kBlockTokens - lo_page + 1;
    const int pg0 = lo_page + split * n_pages / nsplit, pg1 = lo_page + (split + 1) * n_pages / nsplit;
    const int n_tiles = (pg1 - pg0 + kLatPages - 1) / kLatPages;
    if (tid == 0) {
        for (int s = 0; s < stages; s++) mbar_init(&full[s], 1), mbar_init(&empty[s], 8);
        *s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (tid < ROWS) s_m[tid] = -INFINITY, s_l[tid] = 0.f;
    // blocks of 32 pages, a page per lane (tables do not change inside a step)
    int blocks = 0;
    auto lookup = [&](int i) {
        const int pg = pg0 + i * kLatPages + lane;
        blocks = pg < pg1 ? max(page_of(a, sg.seq, pg * kBlockTokens), 0) : 0;
    };
    if (warp == 8) lookup(0);
    __syncthreads();
    if (pdl & 1) griddep_wait();

    float o[MT][NTW][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int n = 0; n < NTW; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[i][n][e] = 0.f;
    if (warp == 8) {
        for (int i = 0; i < n_tiles; i++) {
            const int s = i % stages, pg = pg0 + i * kLatPages, n = min(kLatPages, pg1 - pg), at = i % (32 / kLatPages) * kLatPages;
            if (i > 0 && at == 0) lookup(i);
            const int phys = __shfl_sync(0xffffffffu, blocks, at + lane % kLatPages);
            if (i >= stages && !mbar_wait_bounded(&empty[s], (uint32_t)(i / stages - 1) & 1u, a.status, s_abort)) break;
            if (lane == 0) mbar_expect_tx(&full[s], (uint32_t)n * page_bytes);
            __syncwarp();
            if (lane < n)
                bulk_g2s(ring + ((size_t)s * kLatKeys + lane * kBlockTokens) * LDR, reinterpret_cast<const uint8_t *>(a.kv) + (size_t)phys * page_bytes,
                         page_bytes, &full[s]);
        }
        __syncwarp();
        if (*s_abort)  // a wait ran out: give copies in flight a bounded chance to land before the memory goes
            for (int s = 0; s < stages; s++)
                for (uint32_t k = 0; k < (1u << 12) && !mbar_try_wait(&full[s], 0); k++) {
                }
    } else {
        {  // query rows: q~, then the rotated part, TPR threads per row
            const int r = tid / TPR, j0 = tid % TPR, t = (r0 + r) / H, h = (r0 + r) % H;
            const bool ok = r0 + r < rows;
            const __nv_bfloat16 *qa = reinterpret_cast<const __nv_bfloat16 *>(a.qa) + ((size_t)sg.row0 * H + (ok ? r0 + r : 0)) * KR;
            for (int c = j0 * 8; c < KR; c += TPR * 8) cp_async16(qs + (size_t)r * LDR + c, qa + c, ok);
            asm volatile("cp.async.commit_group;" ::: "memory");
            const __nv_bfloat16 *qr = reinterpret_cast<const __nv_bfloat16 *>(a.q) + (size_t)(sg.row0 + (ok ? t : 0)) * a.ldq + (size_t)h * a.DQ + a.DP;
            const float2 *cs = a.cs + (size_t)(sg.row0 + (ok ? t : 0)) * a.half;
#pragma unroll 4
            for (int j = j0; j < RR; j += TPR) qs[(size_t)r * LDR + KR + j] = __float2bfloat16(ok && j < a.rot_dim ? rotated(qr, cs, a.half, j) : 0.f);
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        named_bar_sync(1, 256);
        // this lane's row and pair of keys when scores become weights: 16 lanes per row, two rows of a warp at a time
        int lo[MT], hi[MT];
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const int r = r0 + warp * 2 * MT + 2 * i + (lane >> 4);
            hi[i] = r < rows ? sg.pos0 + r / H : -1;
            lo[i] = r < rows ? window_first(hi[i], a.window) : 0;
        }
        const float sl = a.scale * 1.4426950408889634f;
        // this warp's k steps, and the query rows' operands for them
        constexpr int NQ = (KR / 16 + kMaxRot / 16 + 7) / 8;
        const int ksteps = (KR + RR) / 16, k_from = warp * ksteps / 8, k_n = (warp + 1) * ksteps / 8 - k_from;
        uint32_t q[NQ][MT][4];
#pragma unroll
        for (int k = 0; k < NQ; k++)
#pragma unroll
            for (int i = 0; i < MT; i++)
                if (k < k_n) ldmatrix_x4(q[k][i], qs + (size_t)(i * 16 + (lane & 15)) * LDR + (lane >> 4) * 8 + (k_from + k) * 16);
        named_bar_sync(1, 256);  // the scores take the query rows' place
        const int end_key = min(last, pg1 * kBlockTokens - 1);
        for (int it = 0; it < n_tiles; it++) {
            const int s = it % stages, kb = (pg0 + it * kLatPages) * kBlockTokens;
            __nv_bfloat16 *ks = ring + (size_t)s * kLatKeys * LDR;
            // when the wait runs out the status word is set: what follows works on whatever is there, and nobody looks at it
            mbar_wait_bounded(&full[s], (uint32_t)(it / stages) & 1u, a.status, s_abort);
            if (kb + kLatKeys - 1 > end_key) {  // nothing is known about what lies behind the last key: its weight is zero, its values must be too
                const int v0 = end_key - kb + 1, per = LDR / 8;
                for (int e = tid; e < (kLatKeys - v0) * per; e += 256) *reinterpret_cast<uint4 *>(ks + (size_t)(v0 + e / per) * LDR + e % per * 8) = make_uint4(0, 0, 0, 0);
            }
            {  // all keys, an eighth of the elements
                float sc[MT][4][4];
#pragma unroll
                for (int i = 0; i < MT; i++)
#pragma unroll
                    for (int e = 0; e < 16; e++) sc[i][e >> 2][e & 3] = 0.f;
                const __nv_bfloat16 *kw = ks + (size_t)(((lane >> 4) << 3) + (lane & 7)) * LDR + ((lane >> 3) & 1) * 8 + k_from * 16;
#pragma unroll
                for (int k = 0; k < NQ; k++) {
                    if (k >= k_n) break;
                    uint32_t b0[4], b1[4];
                    ldmatrix_x4(b0, kw + k * 16);
                    ldmatrix_x4(b1, kw + (size_t)16 * LDR + k * 16);
#pragma unroll
                    for (int i = 0; i < MT; i++) {
                        mma_bf16(sc[i][0], q[k][i], b0[0], b0[1]);
                        mma_bf16(sc[i][1], q[k][i], b0[2], b0[3]);
                        mma_bf16(sc[i][2], q[k][i], b1[0], b1[1]);
                        mma_bf16(sc[i][3], q[k][i], b1[2], b1[3]);
                    }
                }
                float *w = sp + (size_t)warp * ROWS * kLatLS + t2;
#pragma unroll
                for (int i = 0; i < MT; i++)
#pragma unroll
                    for (int e = 0; e < 2; e++)
#pragma unroll
                        for (int c = 0; c < 4; c++)
                            *reinterpret_cast<float2 *>(w + (i * 16 + g + 8 * e) * kLatLS + c * 8) = make_float2(sc[i][c][2 * e], sc[i][c][2 * e + 1]);
            }
            named_bar_sync(1, 256);
#pragma unroll
            for (int i = 0; i < MT; i++) {
                const int r = warp * 2 * MT + 2 * i + (lane >> 4), c = 2 * (lane & 15), key = kb + c, top = min(hi[i], end_key);
                float2 u[8];
#pragma unroll
                for (int k = 0; k < 8; k++) u[k] = *reinterpret_cast<const float2 *>(sp + (k * ROWS + r) * kLatLS + c);
                const float m0 = s_m[r];
#pragma unroll
                for (int k = 4; k >= 1; k >>= 1)
#pragma unroll
                    for (int j = 0; j < 4; j++)
                        if (j < k) u[j].x += u[j + k].x, u[j].y += u[j + k].y;
                const float x0 = key >= lo[i] && key <= top ? u[0].x * sl : -INFINITY, x1 = key + 1 >= lo[i] && key + 1 <= top ? u[0].y * sl : -INFINITY;
                float mx = fmaxf(x0, x1);
#pragma unroll
                for (int off = 8; off >= 1; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
                mx = fmaxf(mx, m0);
                const float ref = mx == -INFINITY ? 0.f : mx, p0 = fast_exp2(x0 - ref), p1 = fast_exp2(x1 - ref);
                uint32_t h2, l2;
                split_pair(p0, p1, h2, l2);
                *reinterpret_cast<uint32_t *>(ph + r * kLatLS + c) = h2, *reinterpret_cast<uint32_t *>(pl + r * kLatLS + c) = l2;
                float sum = p0 + p1;
#pragma unroll
                for (int off = 8; off >= 1; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
                if ((lane & 15) == 0) {
                    const float f = mx == -INFINITY ? 1.f : fast_exp2(m0 - mx);
                    s_m[r] = mx, s_f[r] = f, s_l[r] = s_l[r] * f + sum;
                }
            }
            named_bar_sync(1, 256);
            const __nv_bfloat16 *vw = ks + (size_t)(((lane >> 3) & 1) * 8 + (lane & 7)) * LDR + warp * NTW * 8 + (lane >> 4) * 8;
            const int pw = (lane & 15) * kLatLS + (lane >> 4) * 8;
            bool moved = false;
            float f[MT][2];
#pragma unroll
            for (int i = 0; i < MT; i++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    f[i][e] = s_f[i * 16 + g + 8 * e];
                    moved = moved || f[i][e] != 1.f;
                }
            if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
                for (int i = 0; i < MT; i++)
#pragma unroll
                    for (int n = 0; n < NTW; n++) o[i][n][0] *= f[i][0], o[i][n][1] *= f[i][0], o[i][n][2] *= f[i][1], o[i][n][3] *= f[i][1];
            }
#pragma unroll
            for (int k16 = 0; k16 < kLatKeys / 16; k16++) {
                uint32_t wh[MT][4], wl[MT][4], b[NTW / 2][4];
#pragma unroll
                for (int n = 0; n < NTW / 2; n++) ldmatrix_x4_trans(b[n], vw + (size_t)k16 * 16 * LDR + n * 16);
#pragma unroll
                for (int i = 0; i < MT; i++) {
                    ldmatrix_x4(wh[i], ph + i * 16 * kLatLS + pw + k16 * 16);
                    ldmatrix_x4(wl[i], pl + i * 16 * kLatLS + pw + k16 * 16);
                }
#pragma unroll
                for (int n = 0; n < NTW / 2; n++)
#pragma unroll
                    for (int i = 0; i < MT; i++) {
                        mma_bf16(o[i][2 * n], wh[i], b[n][0], b[n][1]);
                        mma_bf16(o[i][2 * n + 1], wh[i], b[n][2], b[n][3]);
                        mma_bf16(o[i][2 * n], wl[i], b[n][0], b[n][1]);
                        mma_bf16(o[i][2 * n + 1], wl[i], b[n][2], b[n][3]);
                    }
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&empty[s]);  // this warp is done with the stage
        }
    }
    __syncthreads();
    __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(a.qa) + ((size_t)sg.row0 * H + r0) * KR;
    if (nsplit == 1) {
        if (warp == 8) return;
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int r = i * 16 + g + 8 * e;
                if (r0 + r >= rows) continue;
                const float l = s_l[r], f = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
                for (int n = 0; n < NTW; n++)
                    *reinterpret_cast<uint32_t *>(out + (size_t)r * KR + (warp * NTW + n) * 8 + t2) = bf16_pair(o[i][n][2 * e] * f, o[i][n][2 * e + 1] * f);
            }
        return;
    }
    float *mo = reinterpret_cast<float *>(lat_smem);  // [ROWS][KR], in place of the ring
    cluster_wait();                                   // every CTA of the cluster has started: its shared memory may be written
    for (int e = tid; e < ROWS * nsplit; e += kLatThreads) {
        st_cluster_f32(&s_ml[split][e % ROWS][0], (uint32_t)(e / ROWS), s_m[e % ROWS]);
        st_cluster_f32(&s_ml[split][e % ROWS][1], (uint32_t)(e / ROWS), s_l[e % ROWS]);
    }
    if (warp < 8) {
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int e = 0; e < 2; e++)
#pragma unroll
                for (int n = 0; n < NTW; n++)
                    *reinterpret_cast<float2 *>(mo + (size_t)(i * 16 + g + 8 * e) * KR + (warp * NTW + n) * 8 + t2) = make_float2(o[i][n][2 * e], o[i][n][2 * e + 1]);
    }
    cluster_sync();
    // every part's weight per row, then this CTA's share of the columns (the split is 2, 4 or 8)
    const int valid = min(ROWS, rows - r0), cn = KR / nsplit, c0 = split * cn;
    if (tid < ROWS) {
        float ms[8], mx = -INFINITY, sum = 0.f;
#pragma unroll
        for (int s = 0; s < 8; s++) {
            ms[s] = s < nsplit ? s_ml[s][tid][0] : -INFINITY;
            mx = fmaxf(mx, ms[s]);
        }
#pragma unroll
        for (int s = 0; s < 8; s++) {
            ms[s] = ms[s] == -INFINITY ? 0.f : fast_exp2(ms[s] - mx);
            if (s < nsplit) sum += ms[s] * s_ml[s][tid][1];
        }
#pragma unroll
        for (int s = 0; s < 8; s++) sp[s * ROWS + tid] = sum > 0.f ? ms[s] / sum : 0.f;
    }
    __syncthreads();
    for (int e = tid; e < valid * (cn / 4); e += kLatThreads) {
        const int r = e / (cn / 4), c = c0 + e % (cn / 4) * 4;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s0 = 0; s0 < nsplit; s0 += 4) {
            float4 x[4];
#pragma unroll
            for (int s = 0; s < 4; s++) x[s] = s0 + s < nsplit ? ld_cluster_f32x4(mo + (size_t)r * KR + c, (uint32_t)(s0 + s)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int s = 0; s < 4; s++) {
                const float w = sp[(s0 + s) * ROWS + r];
                acc.x = fmaf(w, x[s].x, acc.x), acc.y = fmaf(w, x[s].y, acc.y), acc.z = fmaf(w, x[s].z, acc.z), acc.w = fmaf(w, x[s].w, acc.w);
            }
        }
        *reinterpret_cast<uint2 *>(out + (size_t)r * KR + c) = make_uint2(bf16_pair(acc.x, acc.y), bf16_pair(acc.z, acc.w));
    }
    cluster_sync();  // nobody leaves while its shared memory is being read
}

// ------------------------------------------------------------------------------------------------
// Written out, bf16
// ------------------------------------------------------------------------------------------------
// Page rows of an entry's visible positions, one warp each, into consecutive workspace rows.
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentArgs a, const Seg *__restrict__ segs, const LatentEntry *__restrict__ entries, int pdl) {
    if (pdl & 2) griddep_launch_dependents();
    const LatentEntry en = entries[blockIdx.y];
    const int k = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, n = (a.KR + a.RR) / 8;
    if (pdl & 1) griddep_wait();
    if (k >= en.n_keys) return;
    const int key = en.key0 + k, phys = page_of(a, segs[en.entry].seq, key);
    if (phys < 0) return;
    const uint4 *src = reinterpret_cast<const uint4 *>(reinterpret_cast<const __nv_bfloat16 *>(a.kv) + ((size_t)phys * kBlockTokens + key % kBlockTokens) * a.LDR);
    uint4 *dst = reinterpret_cast<uint4 *>(reinterpret_cast<__nv_bfloat16 *>(a.cx) + (size_t)(en.row0 + k) * (a.KR + a.RR));
    for (int j = lane; j < n; j += 32) dst[j] = src[j];
}

// CTA = 64 query tokens of one head: 4 warps x 16 rows; tiles of 32 keys through two stages (small, for three CTAs on an SM).
constexpr int kTileKeys = 32;
template <int DK, int DV>
__host__ __device__ constexpr size_t latent_tile_smem() { return (size_t)64 * (DK + 8) * 2 + 2 * (size_t)kTileKeys * (DK + DV + 16) * 2; }

template <int DK, int DV>
__global__ void __launch_bounds__(128, DK <= 192 ? 3 : 1) latent_tile_kernel(const LatentArgs a, const Seg *__restrict__ segs, const LatentEntry *__restrict__ entries,
                                                          const int2 *__restrict__ tiles, int pdl) {
    constexpr int LK = DK + 8, LV = DV + 8, CK = DK / 8;
    extern __shared__ __align__(128) uint8_t lat_smem[];
    __nv_bfloat16 *qs = reinterpret_cast<__nv_bfloat16 *>(lat_smem), *kv_s = qs + 64 * LK;  // stages: [K 64 x LK | V 64 x LV]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, h = blockIdx.y;
    if (pdl & 2) griddep_launch_dependents();
    const int2 tile = tiles[blockIdx.x];
    const LatentEntry en = entries[tile.x];
    const Seg sg = segs[en.entry];
    const int nt = min(kLatentTile, sg.T - tile.y), row_base = sg.row0 + tile.y, p0 = sg.pos0 + tile.y, p1 = p0 + nt - 1;
    if (pdl & 1) griddep_wait();
    const __nv_bfloat16 *q = reinterpret_cast<const __nv_bfloat16 *>(a.q) + (size_t)row_base * a.ldq + (size_t)h * a.DQ;
    for (int e = tid; e < 64 * CK; e += 128) {
        const int r = e / CK, c = e % CK * 8;
        if (c < a.DP || c >= a.DP + a.RR) cp_async16(qs + r * LK + c, q + (size_t)(r < nt ? r : 0) * a.ldq + (c < a.DP ? c : 0), r < nt && c < a.DP);
    }
    for (int e = tid; e < 64 * a.RR; e += 128) {
        const int r = e / a.RR, j = e % a.RR;
        qs[r * LK + a.DP + j] =
            __float2bfloat16(r < nt && j < a.rot_dim ? rotated(q + (size_t)r * a.ldq + a.DP, a.cs + (size_t)(row_base + r) * a.half, a.half, j) : 0.f);
    }
    const int start = window_first(p0, a.window) - en.key0;  // workspace index of the first key
    const __nv_bfloat16 *cx = reinterpret_cast<const __nv_bfloat16 *>(a.cx) + (size_t)en.row0 * (a.KR + a.RR) + a.KR;
    const __nv_bfloat16 *kx = reinterpret_cast<const __nv_bfloat16 *>(a.kvx) + (size_t)en.row0 * a.ldx + (size_t)h * a.DP;
    const __nv_bfloat16 *vx = reinterpret_cast<const __nv_bfloat16 *>(a.kvx) + (size_t)en.row0 * a.ldx + (size_t)a.heads * a.DP + (size_t)h * a.DVm;
    const int n_keys = p1 - en.key0 + 1;
    auto load = [&](int stage, int kb) {
        // four threads per key, chunks 4 i + (tid & 3)
        const int j = tid >> 2, key = kb + j;
        const bool in = key < n_keys;
        const size_t row = in ? key : 0;
        __nv_bfloat16 *dk = kv_s + (size_t)stage * kTileKeys * (LK + LV) + j * LK, *dv = kv_s + (size_t)stage * kTileKeys * (LK + LV) + kTileKeys * LK + j * LV;
        const __nv_bfloat16 *kr = kx + row * a.ldx, *rr = cx + row * (a.KR + a.RR), *vr = vx + row * a.ldx;
#pragma unroll
        for (int i = 0; i < DK / 32; i++) {
            const int c = (4 * i + (tid & 3)) * 8;
            const bool ok = in && c < a.DP + a.RR;
            cp_async16(dk + c, c < a.DP ? kr + c : rr + (ok ? c - a.DP : 0), ok);
        }
#pragma unroll
        for (int i = 0; i < DV / 32; i++) {
            const int c = (4 * i + (tid & 3)) * 8;
            const bool ok = in && c < a.DVm;
            cp_async16(dv + c, vr + (ok ? c : 0), ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0, start);
    int lo[2], hi[2], rt[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int r = warp * 16 + g + 8 * e, p = p0 + (r < nt ? r : 0);
        rt[e] = r < nt ? r : -1;
        hi[e] = p - en.key0, lo[e] = window_first(p, a.window) - en.key0;
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    auto qfrag = [&](int kk, uint32_t (&f)[4]) { ldmatrix_x4(f, qs + (size_t)(warp * 16 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8); };
    const float sl = a.scale * 1.4426950408889634f;
    const int vis_lo = window_first(p1, a.window) - en.key0;
    int it = 0;
    for (int kb = start; kb < n_keys; kb += kTileKeys, it++) {
        if (kb + kTileKeys < n_keys) {
            load((it + 1) & 1, kb + kTileKeys);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const __nv_bfloat16 *ks = kv_s + (size_t)(it & 1) * kTileKeys * (LK + LV);
        const bool masked = kb + kTileKeys - 1 > p0 - en.key0 || kb < vis_lo;
        auto kat = [&](int r, int c) { return ks + r * LK + c * 8; };
        auto vat = [&](int r, int c) { return ks + kTileKeys * LK + r * LV + c * 8; };
        attend_tile<DK, DV, kTileKeys, false>(qfrag, kat, vat, kb, masked, lo, hi, 0, sl, m, l, o, lane);
        __syncthreads();
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        if (rt[e] < 0) continue;
        const float f = l[e] > 0.f ? 1.f / l[e] : 0.f;
        __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(a.out) + (size_t)(row_base + rt[e]) * a.ldo + a.out_off + (size_t)h * a.DVm + 2 * (lane & 3);
#pragma unroll
        for (int n = 0; n < DV / 8; n++)
            if (n * 8 < a.DVm) *reinterpret_cast<uint32_t *>(out + n * 8) = bf16_pair(o[n][2 * e] * f, o[n][2 * e + 1] * f);
    }
}

int latent_padded_rank(int kv_rank) { return kv_rank > 0 && kv_rank <= kMaxRank ? (kv_rank + 127) / 128 * 128 : 0; }
int latent_padded_rot(int rot_dim) { return rot_dim > 0 && rot_dim <= kMaxRot ? (rot_dim + 15) / 16 * 16 : 0; }

// Head sizes of the written-out form: the smallest of these that holds both.
struct TileSize {
    int dk, dv;
};
constexpr TileSize kTileSizes[] = {{64, 64}, {128, 64}, {128, 128}, {192, 128}, {256, 128}, {256, 256}};
static int tile_size(int dp, int rr, int dv) {
    for (int i = 0; i < 6; i++)
        if (dp + rr <= kTileSizes[i].dk && dv <= kTileSizes[i].dv) return i;
    return -1;
}
bool latent_expandable(int dim, int rot_dim, int vdim) { return tile_size((dim + 7) / 8 * 8, latent_padded_rot(rot_dim), (vdim + 7) / 8 * 8) >= 0; }

template <class... P, class... Args>
static int32_t launch(void (*kern)(P...), dim3 grid, int threads, size_t smem, int cluster, int pdl, cudaStream_t st, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[2];
    int na = 0;
    if (pdl & 1) {
        attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[na++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (cluster > 1) {
        attr[na].id = cudaLaunchAttributeClusterDimension;
        attr[na].val.clusterDim.x = (unsigned)cluster, attr[na].val.clusterDim.y = 1, attr[na].val.clusterDim.z = 1;
        na++;
    }
    cfg.gridDim = grid, cfg.blockDim = dim3((unsigned)threads), cfg.dynamicSmemBytes = smem, cfg.stream = st, cfg.attrs = attr, cfg.numAttrs = (unsigned)na;
    JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, kern, args...));
    return JGPT_OK;
}

template <class K>
static int32_t opt_in(K kern, size_t smem, int &set_for) {
    int dev = 0;
    JGPT_CUDA_TRY(cudaGetDevice(&dev));
    if (set_for != dev) {
        JGPT_CUDA_TRY(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        set_for = dev;
    }
    return JGPT_OK;
}

int32_t launch_latent_prep(bool f32, const StepDesc &d, const LatentArgs &a, int pdl, cudaStream_t st) {
    const int items = d.rows * (a.own_cache ? 2 : 1), warps = items <= 4 * a.sm_count ? 2 : 8;
    const dim3 grid((unsigned)((items + warps - 1) / warps));
    if (f32) return launch(latent_prep_kernel<float>, grid, 32 * warps, 0, 1, pdl, st, a, d.seq, d.pos, d.rows, pdl);
    return launch(latent_prep_kernel<__nv_bfloat16>, grid, 32 * warps, 0, 1, pdl, st, a, d.seq, d.pos, d.rows, pdl);
}

template <int NTW, int MT>
static int32_t attn_run(const StepDesc &d, const LatentArgs &a, const Seg *list, int n, int max_rows, bool single, int pdl, cudaStream_t st) {
    auto kern = latent_attn_kernel<NTW, MT>;
    static thread_local int set_for = -1;
    if (int32_t rc = opt_in(kern, kMaxSmem, set_for)) return rc;
    const size_t fixed = latent_fixed_smem<MT>(a.LDR), stage = (size_t)kLatKeys * a.LDR * 2;
    const size_t room = MT == 1 ? kMaxSmem / 2 : kMaxSmem;  // two CTAs of 16 rows share an SM
    const int stages = (int)std::min<size_t>(6, (std::max(room, fixed + 2 * stage) - fixed) / stage), blocks = (max_rows + 16 * MT - 1) / (16 * MT);
    JGPT_REQUIRE(stages >= 2 && fixed + stages * stage <= kMaxSmem, JGPT_ERR_UNSUPPORTED, "latent of %d, rotated part of %d", a.KR, a.RR);
    int split = 1;
    if (single) {  // the grid stays within what the SMs hold, every CTA keeps two tiles
        const int keys = a.window > 0 ? std::min(a.window, d.max_len) : d.max_len, tiles = keys / kLatKeys + 1;
        while (split < 8 && n * blocks * split * 2 <= (MT == 1 ? 2 : 1) * a.sm_count && tiles >= split * 2 * 2) split *= 2;
    }
    const dim3 grid((unsigned)split, (unsigned)blocks, (unsigned)n);
    return launch(kern, grid, kLatThreads, fixed + stages * stage, split, pdl, st, a, list, stages, pdl);
}

template <int NTW>
static int32_t attn_rows(const StepDesc &d, const LatentArgs &a, const Seg *list, int n, int max_rows, bool single, int pdl, cudaStream_t st) {
    return max_rows <= 16 ? attn_run<NTW, 1>(d, a, list, n, max_rows, single, pdl, st) : attn_run<NTW, 2>(d, a, list, n, max_rows, single, pdl, st);
}

int32_t launch_latent_attention(bool f32, const StepDesc &d, const LatentArgs &a, int pdl, cudaStream_t st) {
    if (f32) {
        latent_rows_kernel<float><<<(unsigned)((d.rows * (long long)a.heads + 7) / 8), 256, 0, st>>>(a, d.seq, d.pos, d.rows);
        JGPT_CUDA_TRY(cudaGetLastError());
        return JGPT_OK;
    }
    auto run = [&](const Seg *list, int n, int max_rows, bool single) -> int32_t {
        switch (a.KR) {
            case 128: return attn_rows<2>(d, a, list, n, max_rows, single, pdl, st);
            case 256: return attn_rows<4>(d, a, list, n, max_rows, single, pdl, st);
            case 384: return attn_rows<6>(d, a, list, n, max_rows, single, pdl, st);
            case 512: return attn_rows<8>(d, a, list, n, max_rows, single, pdl, st);
        }
        return fail(JGPT_ERR_UNSUPPORTED, "latent of %d", a.KR);
    };
    if (d.n_singles)
        if (int32_t rc = run(d.lat_singles, d.n_singles, a.heads, true)) return rc;
    return d.n_lat_short ? run(d.lat_short, d.n_lat_short, d.lat_short_max * a.heads, false) : JGPT_OK;
}

int32_t launch_latent_gather(const StepDesc &d, const LatentArgs &a, int first, int n, int max_keys, int pdl, cudaStream_t st) {
    return launch(latent_gather_kernel, dim3((unsigned)((max_keys + 7) / 8), (unsigned)n), 256, 0, 1, pdl, st, a, d.segs, d.lat_long + first, pdl);
}

template <int DK, int DV>
static int32_t tile_run(const StepDesc &d, const LatentArgs &a, int first, int n, int pdl, cudaStream_t st) {
    auto kern = latent_tile_kernel<DK, DV>;
    static thread_local int set_for = -1;
    if (int32_t rc = opt_in(kern, latent_tile_smem<DK, DV>(), set_for)) return rc;
    return launch(kern, dim3((unsigned)n, (unsigned)a.heads), 128, latent_tile_smem<DK, DV>(), 1, pdl, st, a, d.segs, d.lat_long, d.lat_tiles + first, pdl);
}

int32_t launch_latent_tiles(const StepDesc &d, const LatentArgs &a, int first_tile, int n_tiles, int pdl, cudaStream_t st) {
    switch (tile_size(a.DP, a.RR, a.DVm)) {
        case 0: return tile_run<64, 64>(d, a, first_tile, n_tiles, pdl, st);
        case 1: return tile_run<128, 64>(d, a, first_tile, n_tiles, pdl, st);
        case 2: return tile_run<128, 128>(d, a, first_tile, n_tiles, pdl, st);
        case 3: return tile_run<192, 128>(d, a, first_tile, n_tiles, pdl, st);
        case 4: return tile_run<256, 128>(d, a, first_tile, n_tiles, pdl, st);
        case 5: return tile_run<256, 256>(d, a, first_tile, n_tiles, pdl, st);
    }
    return fail(JGPT_ERR_UNSUPPORTED, "head sizes %d + %d / %d", a.DP, a.RR, a.DVm);
}

}  // namespace mix
}  // namespace jgpt
