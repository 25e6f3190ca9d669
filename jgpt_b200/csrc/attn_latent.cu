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

// One warp per (row, part): part 0 the query latent, part 1 the key latent and the rotated part.
template <class AT>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int rows, int pdl) {
    const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, parts = a.own_cache ? 2 : 1;
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    if (item >= rows * parts) return;
    const int r = item / parts, part = item % parts;
    const AT *proj = reinterpret_cast<const AT *>(a.proj) + (size_t)r * a.ldp;
    const AT *src = proj + (part ? a.c_off : a.dq_off);
    const float *gamma = part ? a.dkv_norm : a.dq_norm;
    const int n = part ? a.kv_rank : a.q_rank, padded = part ? a.KR : a.ldcq;
    float ss = 0.f;
    for (int j = lane; j < n; j += 32) {
        const float v = act_load(src + j);
        ss += v * v;
    }
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    const float inv = 1.f / sqrtf(ss / (float)n + a.eps);
    AT *dst = reinterpret_cast<AT *>(a.cq) + (size_t)r * a.ldcq;
    if (part) {
        const int phys = page_of(a, seq[r], pos[r]);
        if (phys < 0) return;
        dst = reinterpret_cast<AT *>(a.kv) + ((size_t)phys * kBlockTokens + pos[r] % kBlockTokens) * a.LDR;
    }
    for (int j = lane; j < padded; j += 32) act_store(dst + j, j < n ? act_load(src + j) * inv * gamma[j] : 0.f);
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
// CTA = 16 MT (token, head) rows of an entry, eight warps, tiles of 64 keys = four pages brought in by bulk copies (a page is
// contiguous, its row stride an odd number of 16-byte units, so ldmatrix is free of bank conflicts).  A warp scores eight keys
// of a tile for all rows; the row maxima and the weights (bf16 high and low parts) meet in shared memory; then a warp adds up
// its eighth of the latent's columns.  A cluster splits the keys; partial sums meet through cluster shared memory.
constexpr int kLatKeys = 64, kLatPages = kLatKeys / kBlockTokens, kLatLP = kLatKeys + 8;
constexpr size_t kMaxSmem = 232448;

template <int MT>
__host__ __device__ constexpr size_t latent_fixed_smem(int LDR) {
    return (size_t)16 * MT * LDR * 2 + 2 * (size_t)16 * MT * kLatLP * 2 + sizeof(float) * 8 * 16 * MT;
}

template <int NTW, int MT>
__global__ void __launch_bounds__(256, 1) latent_attn_kernel(const LatentArgs a, const Seg *__restrict__ segs, const int *__restrict__ list, int stages, int pdl) {
    constexpr int KR = NTW * 64, ROWS = 16 * MT, MAXST = 8;
    extern __shared__ __align__(128) uint8_t lat_smem[];
    __shared__ __align__(8) uint64_t full[MAXST];
    __shared__ int s_abort_mem;
    volatile int *s_abort = &s_abort_mem;
    const int LDR = a.LDR, RR = a.RR, H = a.heads;
    const uint32_t page_bytes = (uint32_t)(kBlockTokens * LDR * 2);
    __nv_bfloat16 *ring = reinterpret_cast<__nv_bfloat16 *>(lat_smem);  // [stages][64][LDR]
    __nv_bfloat16 *qs = ring + (size_t)stages * kLatKeys * LDR;         // [ROWS][LDR]
    __nv_bfloat16 *ph = qs + (size_t)ROWS * LDR, *pl = ph + ROWS * kLatLP;
    float *red = reinterpret_cast<float *>(pl + ROWS * kLatLP);         // [8][ROWS]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = 2 * (lane & 3);
    const int nsplit = gridDim.x, split = blockIdx.x, r0 = blockIdx.y * ROWS;
    if (pdl & 2) griddep_launch_dependents();
    const Seg sg = segs[list[blockIdx.z]];
    const int rows = sg.T * H;
    if (r0 >= rows) return;
    const int first = window_first(sg.pos0 + r0 / H, a.window), last = sg.pos0 + min(rows - 1, r0 + ROWS - 1) / H;
    const int lo_page = first / kBlockTokens, n_pages = last / kBlockTokens - lo_page + 1;
    const int pg0 = lo_page + split * n_pages / nsplit, pg1 = lo_page + (split + 1) * n_pages / nsplit;
    const int n_tiles = (pg1 - pg0 + kLatPages - 1) / kLatPages;
    if (tid == 0) {
        for (int s = 0; s < stages; s++) mbar_init(&full[s], 1);
        *s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    if (pdl & 1) griddep_wait();

    // warp 0 brings tiles in: lanes 0-3 a page each, its block looked up a tile ahead
    int phys = 0;
    auto lookup = [&](int i) {
        const int pg = pg0 + i * kLatPages + lane;
        phys = lane < kLatPages && pg < pg1 ? max(page_of(a, sg.seq, pg * kBlockTokens), 0) : 0;
    };
    auto fetch = [&](int i) {
        const int s = i % stages, pg = pg0 + i * kLatPages, n = min(kLatPages, pg1 - pg);
        if (lane == 0) mbar_expect_tx(&full[s], (uint32_t)n * page_bytes);
        __syncwarp();
        if (lane < n)
            bulk_g2s(ring + ((size_t)s * kLatKeys + lane * kBlockTokens) * LDR, reinterpret_cast<const uint8_t *>(a.kv) + (size_t)phys * page_bytes, page_bytes,
                     &full[s]);
        lookup(i + 1);
    };
    int issued = 0;
    if (warp == 0) {
        lookup(0);
        for (; issued < stages && issued < n_tiles; issued++) fetch(issued);
    }
    {  // query rows: q~, then the rotated part
        const __nv_bfloat16 *qa = reinterpret_cast<const __nv_bfloat16 *>(a.qa) + (size_t)sg.row0 * H * KR;
        for (int e = tid; e < ROWS * (KR / 8); e += 256) {
            const int r = e / (KR / 8), c = e % (KR / 8) * 8;
            const bool ok = r0 + r < rows;
            cp_async16(qs + (size_t)r * LDR + c, qa + (size_t)(ok ? r0 + r : 0) * KR + c, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        for (int e = tid; e < ROWS * RR; e += 256) {
            const int r = e / RR, j = e % RR, t = (r0 + r) / H, h = (r0 + r) % H;
            float v = 0.f;
            if (r0 + r < rows && j < a.rot_dim)
                v = rotated(reinterpret_cast<const __nv_bfloat16 *>(a.q) + (size_t)(sg.row0 + t) * a.ldq + (size_t)h * a.DQ + a.DP,
                            a.cs + (size_t)(sg.row0 + t) * a.half, a.half, j);
            qs[(size_t)r * LDR + KR + j] = __float2bfloat16(v);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();

    int lo[MT][2], hi[MT][2];
    float m[MT][2], l[MT][2], o[MT][NTW][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int r = r0 + i * 16 + g + 8 * e;
            hi[i][e] = r < rows ? sg.pos0 + r / H : -1;
            lo[i][e] = r < rows ? window_first(hi[i][e], a.window) : 0;
            m[i][e] = -INFINITY, l[i][e] = 0.f;
        }
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int n = 0; n < NTW; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[i][n][e] = 0.f;
    const float sl = a.scale * 1.4426950408889634f;
    const int ksteps = (KR + RR) / 16, end_key = min(last, pg1 * kBlockTokens - 1);
    bool failed = false;
    for (int it = 0; it < n_tiles; it++) {
        const int s = it % stages, kb = (pg0 + it * kLatPages) * kBlockTokens;
        __nv_bfloat16 *ks = ring + (size_t)s * kLatKeys * LDR;
        const bool ok = mbar_wait_bounded(&full[s], (uint32_t)(it / stages) & 1u, a.status, s_abort);
        if (kb + kLatKeys - 1 > end_key) {  // nothing is known about what lies behind the last key: its weight is zero, its values must be too
            const int v0 = end_key - kb + 1, per = LDR / 8;
            for (int e = tid; e < (kLatKeys - v0) * per; e += 256) *reinterpret_cast<uint4 *>(ks + (size_t)(v0 + e / per) * LDR + e % per * 8) = make_uint4(0, 0, 0, 0);
        }
        float sc[MT][4];
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) sc[i][e] = 0.f;
        const __nv_bfloat16 *kw = ks + (size_t)(warp * 8 + (lane & 7)) * LDR + (lane >> 3) * 8, *qw = qs + (size_t)(lane & 15) * LDR + (lane >> 4) * 8;
        auto score = [&](int kk, uint32_t b0, uint32_t b1) {
#pragma unroll
            for (int i = 0; i < MT; i++) {
                uint32_t q[4];
                ldmatrix_x4(q, qw + (size_t)i * 16 * LDR + kk * 16);
                mma_bf16(sc[i], q, b0, b1);
            }
        };
        int kk = 0;
#pragma unroll 4
        for (; kk + 1 < ksteps; kk += 2) {
            uint32_t b[4];
            ldmatrix_x4(b, kw + kk * 16);
            score(kk, b[0], b[1]);
            score(kk + 1, b[2], b[3]);
        }
        if (kk < ksteps) {  // the upper two matrices would lie past the row: their lanes read the lower ones again
            uint32_t b[4];
            ldmatrix_x4(b, kw + kk * 16 - (lane >= 16 ? 16 : 0));
            score(kk, b[0], b[1]);
        }
        const int key = kb + warp * 8 + t2;
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                float mx = -INFINITY;
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    float &x = sc[i][2 * e + c];
                    x = key + c >= lo[i][e] && key + c <= min(hi[i][e], end_key) ? x * sl : -INFINITY;
                    mx = fmaxf(mx, x);
                }
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                if ((lane & 3) == 0) red[warp * ROWS + i * 16 + g + 8 * e] = mx;
            }
        if (__syncthreads_or(!ok)) {
            failed = true;
            break;
        }
        float f[MT][2];
        bool moved = false;
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                float mn = m[i][e];
#pragma unroll
                for (int w = 0; w < 8; w++) mn = fmaxf(mn, red[w * ROWS + i * 16 + g + 8 * e]);
                f[i][e] = mn == -INFINITY ? 1.f : fast_exp2(m[i][e] - mn);
                m[i][e] = mn;
                const float ref = mn == -INFINITY ? 0.f : mn;
                const float p0 = fast_exp2(sc[i][2 * e] - ref), p1 = fast_exp2(sc[i][2 * e + 1] - ref);
                l[i][e] = l[i][e] * f[i][e] + p0 + p1;
                moved = moved || f[i][e] != 1.f;
                uint32_t h2, l2;
                split_pair(p0, p1, h2, l2);
                const int at = (i * 16 + g + 8 * e) * kLatLP + warp * 8 + t2;
                *reinterpret_cast<uint32_t *>(ph + at) = h2, *reinterpret_cast<uint32_t *>(pl + at) = l2;
            }
        __syncthreads();
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int i = 0; i < MT; i++)
#pragma unroll
                for (int n = 0; n < NTW; n++) o[i][n][0] *= f[i][0], o[i][n][1] *= f[i][0], o[i][n][2] *= f[i][1], o[i][n][3] *= f[i][1];
        }
        const __nv_bfloat16 *vw = ks + (size_t)(((lane >> 3) & 1) * 8 + (lane & 7)) * LDR + warp * NTW * 8 + (lane >> 4) * 8;
        const int pw = (lane & 15) * kLatLP + (lane >> 4) * 8;
#pragma unroll
        for (int k16 = 0; k16 < kLatKeys / 16; k16++) {
            uint32_t wh[MT][4], wl[MT][4];
#pragma unroll
            for (int i = 0; i < MT; i++) {
                ldmatrix_x4(wh[i], ph + i * 16 * kLatLP + pw + k16 * 16);
                ldmatrix_x4(wl[i], pl + i * 16 * kLatLP + pw + k16 * 16);
            }
#pragma unroll
            for (int n = 0; n < NTW; n += 2) {
                uint32_t b[4];
                ldmatrix_x4_trans(b, vw + (size_t)k16 * 16 * LDR + n * 8);
#pragma unroll
                for (int i = 0; i < MT; i++) {
                    mma_bf16(o[i][n], wh[i], b[0], b[1]);
                    mma_bf16(o[i][n], wl[i], b[0], b[1]);
                    mma_bf16(o[i][n + 1], wh[i], b[2], b[3]);
                    mma_bf16(o[i][n + 1], wl[i], b[2], b[3]);
                }
            }
        }
        __syncthreads();  // the stage, the maxima and the weights are free
        if (warp == 0 && issued < n_tiles) fetch(issued++);
    }
    if (failed) {  // give copies in flight a bounded chance to land, then leave together
        if (tid == 0)
            for (int i = 0; i < stages; i++)
                for (uint32_t k = 0; k < (1u << 16) && !mbar_try_wait(&full[i], (uint32_t)((n_tiles - 1 - i) / stages) & 1u); k++) {
                }
        __syncthreads();
        return;
    }
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            l[i][e] += __shfl_xor_sync(0xffffffffu, l[i][e], 1);
            l[i][e] += __shfl_xor_sync(0xffffffffu, l[i][e], 2);
            if ((lane & 3) == 0) red[warp * ROWS + i * 16 + g + 8 * e] = l[i][e];
        }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            l[i][e] = 0.f;
#pragma unroll
            for (int w = 0; w < 8; w++) l[i][e] += red[w * ROWS + i * 16 + g + 8 * e];
        }
    __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(a.qa) + ((size_t)sg.row0 * H + r0) * KR;
    if (nsplit == 1) {
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int r = i * 16 + g + 8 * e;
                if (r0 + r >= rows) continue;
                const float f = l[i][e] > 0.f ? 1.f / l[i][e] : 0.f;
#pragma unroll
                for (int n = 0; n < NTW; n++)
                    *reinterpret_cast<uint32_t *>(out + (size_t)r * KR + (warp * NTW + n) * 8 + t2) = bf16_pair(o[i][n][2 * e] * f, o[i][n][2 * e + 1] * f);
            }
        return;
    }
    float *mo = reinterpret_cast<float *>(lat_smem), *ml = mo + (size_t)ROWS * KR;  // [ROWS][KR], [ROWS][m, l], in place of the ring
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int r = i * 16 + g + 8 * e;
            if (warp == 0 && (lane & 3) == 0) ml[2 * r] = m[i][e], ml[2 * r + 1] = l[i][e];
#pragma unroll
            for (int n = 0; n < NTW; n++)
                *reinterpret_cast<float2 *>(mo + (size_t)r * KR + (warp * NTW + n) * 8 + t2) = make_float2(o[i][n][2 * e], o[i][n][2 * e + 1]);
        }
    cluster_sync();
    const int valid = min(ROWS, rows - r0), c0 = split * KR / nsplit, cn = (split + 1) * KR / nsplit - c0;
    for (int e = tid; e < valid * cn; e += 256) {
        const int r = e / cn, c = c0 + e % cn;
        float mx = -INFINITY, sum = 0.f, acc = 0.f;
        for (int s = 0; s < nsplit; s++) mx = fmaxf(mx, ld_cluster_f32(ml + 2 * r, (uint32_t)s));
        for (int s = 0; s < nsplit; s++) {
            const float ms = ld_cluster_f32(ml + 2 * r, (uint32_t)s), f = ms == -INFINITY ? 0.f : fast_exp2(ms - mx);
            sum += f * ld_cluster_f32(ml + 2 * r + 1, (uint32_t)s), acc += f * ld_cluster_f32(mo + (size_t)r * KR + c, (uint32_t)s);
        }
        out[(size_t)r * KR + c] = __float2bfloat16(sum > 0.f ? acc / sum : 0.f);
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

// CTA = 64 query tokens of one head: 4 warps x 16 rows; tiles of 64 keys through two stages.
template <int DK, int DV>
__host__ __device__ constexpr size_t latent_tile_smem() { return (size_t)64 * (DK + 8) * 2 + 2 * (size_t)kLatKeys * (DK + DV + 16) * 2; }

template <int DK, int DV>
__global__ void __launch_bounds__(128) latent_tile_kernel(const LatentArgs a, const Seg *__restrict__ segs, const LatentEntry *__restrict__ entries,
                                                          const int2 *__restrict__ tiles, int pdl) {
    constexpr int LK = DK + 8, LV = DV + 8, CK = DK / 8, CV = DV / 8;
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
        __nv_bfloat16 *dk = kv_s + (size_t)stage * kLatKeys * (LK + LV), *dv = dk + kLatKeys * LK;
        for (int e = tid; e < kLatKeys * (CK + CV); e += 128) {
            const int j = e / (CK + CV), x = e % (CK + CV), key = kb + j;
            const bool in = key < n_keys;
            const size_t row = in ? key : 0;
            if (x < CK) {
                const int c = x * 8;
                const bool rot = c >= a.DP;
                const bool ok = in && c < a.DP + a.RR;
                cp_async16(dk + j * LK + c, rot ? cx + row * (a.KR + a.RR) + (ok ? c - a.DP : 0) : kx + row * a.ldx + c, ok);
            } else {
                const int c = (x - CK) * 8;
                const bool ok = in && c < a.DVm;
                cp_async16(dv + j * LV + c, vx + row * a.ldx + (ok ? c : 0), ok);
            }
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
    for (int kb = start; kb < n_keys; kb += kLatKeys, it++) {
        if (kb + kLatKeys < n_keys) {
            load((it + 1) & 1, kb + kLatKeys);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const __nv_bfloat16 *ks = kv_s + (size_t)(it & 1) * kLatKeys * (LK + LV);
        const bool masked = kb + kLatKeys - 1 > p0 - en.key0 || kb < vis_lo;
        attend_tile<DK, DV, kLatKeys>(qfrag, ks, ks + kLatKeys * LK, kb, masked, lo, hi, sl, m, l, o, lane);
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
    const dim3 grid((unsigned)((d.rows * (a.own_cache ? 2 : 1) + 7) / 8));
    if (f32) return launch(latent_prep_kernel<float>, grid, 256, 0, 1, pdl, st, a, d.seq, d.pos, d.rows, pdl);
    return launch(latent_prep_kernel<__nv_bfloat16>, grid, 256, 0, 1, pdl, st, a, d.seq, d.pos, d.rows, pdl);
}

template <int NTW, int MT>
static int32_t attn_run(const StepDesc &d, const LatentArgs &a, const int *list, int n, int max_rows, bool single, int pdl, cudaStream_t st) {
    auto kern = latent_attn_kernel<NTW, MT>;
    static thread_local int set_for = -1;
    if (int32_t rc = opt_in(kern, kMaxSmem - 1024, set_for)) return rc;
    const size_t fixed = latent_fixed_smem<MT>(a.LDR), stage = (size_t)kLatKeys * a.LDR * 2;
    const int stages = (int)std::min<size_t>(4, (kMaxSmem - 1024 - fixed) / stage), blocks = (max_rows + 16 * MT - 1) / (16 * MT);
    JGPT_REQUIRE(stages >= 2, JGPT_ERR_UNSUPPORTED, "latent of %d, rotated part of %d", a.KR, a.RR);
    int split = 1;
    if (single) {  // the grid stays within one CTA per SM, every CTA keeps two tiles
        const int keys = a.window > 0 ? std::min(a.window, d.max_len) : d.max_len, tiles = keys / kLatKeys + 1;
        while (split < 8 && n * blocks * split * 2 <= a.sm_count && tiles >= split * 2 * 2) split *= 2;
    }
    const dim3 grid((unsigned)split, (unsigned)blocks, (unsigned)n);
    return launch(kern, grid, 256, fixed + stages * stage, split, pdl, st, a, d.segs, list, stages, pdl);
}

template <int NTW>
static int32_t attn_rows(const StepDesc &d, const LatentArgs &a, const int *list, int n, int max_rows, bool single, int pdl, cudaStream_t st) {
    return max_rows <= 16 ? attn_run<NTW, 1>(d, a, list, n, max_rows, single, pdl, st) : attn_run<NTW, 2>(d, a, list, n, max_rows, single, pdl, st);
}

int32_t launch_latent_attention(bool f32, const StepDesc &d, const LatentArgs &a, int pdl, cudaStream_t st) {
    if (f32) {
        latent_rows_kernel<float><<<(unsigned)((d.rows * (long long)a.heads + 7) / 8), 256, 0, st>>>(a, d.seq, d.pos, d.rows);
        JGPT_CUDA_TRY(cudaGetLastError());
        return JGPT_OK;
    }
    auto run = [&](const int *list, int n, int max_rows, bool single) -> int32_t {
        switch (a.KR) {
            case 128: return attn_rows<2>(d, a, list, n, max_rows, single, pdl, st);
            case 256: return attn_rows<4>(d, a, list, n, max_rows, single, pdl, st);
            case 384: return attn_rows<6>(d, a, list, n, max_rows, single, pdl, st);
            case 512: return attn_rows<8>(d, a, list, n, max_rows, single, pdl, st);
        }
        return fail(JGPT_ERR_UNSUPPORTED, "latent of %d", a.KR);
    };
    if (d.n_singles)
        if (int32_t rc = run(d.singles, d.n_singles, a.heads, true)) return rc;
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
