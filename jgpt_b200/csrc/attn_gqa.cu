// Paged attention of the layered decoder: query heads in groups that share a key head, head sizes up to 256 (padded to what
// the kernels are built for), all earlier positions or those of the query's chunk, optional norms and rotation of the heads,
// one or two maps per head (mixers.cuh), an optional output gate per head or per element.
//
//   attn_prep_kernel     query heads normed and rotated in place, keys likewise and values into the pages
//   attn_rows_kernel     one warp per (row, head), fp32: the exact mode
//   attn_tile_kernel     portions of prompts, bf16 tensor cores
//   attn_single_kernel   single tokens, bf16 tensor cores over a split sequence, with the preparation of its own heads
#include "mixers.cuh"

#include <algorithm>

#include "attn_mma.cuh"

namespace jgpt {
namespace mix {

__host__ __device__ __forceinline__ int first_visible(int pos, int chunk) { return chunk > 0 ? pos / chunk * chunk : 0; }

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// A head (map) of a row in the 8-element pieces of `lanes` neighbouring lanes (a power of two; every lane of the warp takes
// part): norm over its dim elements, rotation.  buf: 8 floats per lane of the group.
__device__ __forceinline__ void prepare_head(float (&x)[8], int piece, int lanes, int dim, const float *w, float eps, const float2 *cs, int half,
                                             int interleaved, float *buf) {
    const int j0 = piece * 8;
    if (w) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; e++) ss += x[e] * x[e];
        for (int off = lanes >> 1; off >= 1; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
        const float inv = 1.f / sqrtf(ss / (float)dim + eps);
#pragma unroll
        for (int e = 0; e < 8; e++) x[e] = j0 + e < dim ? x[e] * inv * __ldg(w + j0 + e) : 0.f;
    }
    if (!half) return;
    if (interleaved) {
#pragma unroll
        for (int e = 0; e < 8; e += 2)
            if (j0 + e < 2 * half) {
                const float2 t = __ldg(cs + ((j0 + e) >> 1));
                const float u = x[e], v = x[e + 1];
                x[e] = u * t.x - v * t.y, x[e + 1] = v * t.x + u * t.y;
            }
        return;
    }
#pragma unroll
    for (int e = 0; e < 8; e++) buf[j0 + e] = x[e];
    __syncwarp();
#pragma unroll
    for (int e = 0; e < 8; e++) {
        const int j = j0 + e;
        if (j >= 2 * half) continue;
        const float2 t = __ldg(cs + (j < half ? j : j - half));
        x[e] = j < half ? x[e] * t.x - buf[j + half] * t.y : x[e] * t.x + buf[j - half] * t.y;
    }
    __syncwarp();
}
__host__ __device__ __forceinline__ int head_lanes(int DK) { return DK <= 32 ? 4 : (DK <= 64 ? 8 : (DK <= 128 ? 16 : 32)); }

// Vectors of a row: its query maps (when they are prepared), key maps, values; a vector per head_lanes(DK) lanes.
template <class AT>
__global__ void __launch_bounds__(256) attn_prep_kernel(const AttnArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int rows, int pdl) {
    __shared__ float bufs[256 * 8];
    if (pdl & 2) griddep_launch_dependents();
    const int lanes = head_lanes(a.DK), nq = a.prepared() ? a.heads * a.maps : 0, nk = a.kv_heads * a.maps, nv = nq + nk + a.kv_heads;
    const long long item = ((long long)blockIdx.x * 256 + threadIdx.x) / lanes;
    const bool ok = item < (long long)rows * nv;
    const int r = ok ? (int)(item / nv) : 0, i = ok ? (int)(item % nv) : 0, piece = threadIdx.x & (lanes - 1);
    if (pdl & 1) griddep_wait();
    AT *proj = reinterpret_cast<AT *>(a.proj) + (size_t)r * a.ldp;
    const int p = pos[r];
    AT *page = nullptr;
    if (i >= nq) {
        const int phys = page_of(a, seq[r], p), g = i < nq + nk ? (i - nq) / a.maps : i - nq - nk;
        if (phys >= 0) page = reinterpret_cast<AT *>(a.kv) + ((size_t)phys * a.kv_heads + g) * a.page_head();
    }
    const bool value = i >= nq + nk, mine = ok && (i < nq || page);
    if (value && mine) {
        const AT *src = proj + a.v_off + (i - nq - nk) * a.DV;
        AT *dst = page + kBlockTokens * a.maps * a.DK + (size_t)(p % kBlockTokens) * a.DV;
        constexpr int E = 16 / sizeof(AT);
        for (int c = piece * E; c < a.DV; c += lanes * E) *reinterpret_cast<uint4 *>(dst + c) = *reinterpret_cast<const uint4 *>(src + c);
    }
    float x[8];
    AT *src = proj + (i < nq ? a.q_off + i * a.DK : a.k_off + (i - nq) * a.DK) + piece * 8;
    const bool load = mine && !value && piece * 8 < a.DK;
    if (load) load8(src, x);
    else {
#pragma unroll
        for (int e = 0; e < 8; e++) x[e] = 0.f;
    }
    if (a.prepared())
        prepare_head(x, piece, lanes, a.dim, i < nq ? a.q_norm : a.k_norm, a.eps, a.cs + (size_t)r * a.half, a.half, a.interleaved, bufs + (threadIdx.x - piece) * 8);
    if (!load) return;
    if (i < nq) store8(src, x);
    else store8(page + (size_t)(p % kBlockTokens) * a.maps * a.DK + (i - nq) % a.maps * a.DK + piece * 8, x);
}

// One warp per (row, query head): lane l holds elements l, l + 32, ... of q and of the output.
template <class AT>
__global__ void __launch_bounds__(256) attn_rows_kernel(const AttnArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int rows) {
    constexpr int MAXE = 8;
    const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= rows * a.heads) return;
    const int r = item / a.heads, h = item % a.heads, g = h / (a.heads / a.kv_heads), nk = a.DK / 32, nv = a.DV / 32, kw = a.maps * a.DK;
    const AT *proj = reinterpret_cast<const AT *>(a.proj) + (size_t)r * a.ldp;
    float first[MAXE], o[MAXE], f = 1.f;
    const int p = pos[r], s = seq[r];
    for (int map = 0; map < a.maps; map++) {
        float q[MAXE], m = -INFINITY, l = 0.f;
#pragma unroll
        for (int e = 0; e < MAXE; e++)
            q[e] = e < nk ? act_load(proj + a.q_off + (h * a.maps + map) * a.DK + lane + 32 * e) * a.scale : 0.f, first[e] = map ? o[e] * f : 0.f, o[e] = 0.f;
        for (int j = first_visible(p, a.chunk); j <= p; j++) {
            const int phys = page_of(a, s, j);
            if (phys < 0) break;
            const AT *k = reinterpret_cast<const AT *>(a.kv) + ((size_t)phys * a.kv_heads + g) * a.page_head();
            const AT *v = k + kBlockTokens * kw + (size_t)(j % kBlockTokens) * a.DV + lane;
            k += (size_t)(j % kBlockTokens) * kw + map * a.DK + lane;
            float d = 0.f;
#pragma unroll
            for (int e = 0; e < MAXE; e++)
                if (e < nk) d = fmaf(q[e], act_load(k + 32 * e), d);
#pragma unroll
            for (int off = 16; off >= 1; off >>= 1) d += __shfl_xor_sync(0xffffffffu, d, off);
            const float mn = fmaxf(m, d), fo = expf(m - mn), w = expf(d - mn);
            m = mn, l = l * fo + w;
#pragma unroll
            for (int e = 0; e < MAXE; e++)
                if (e < nv) o[e] = fmaf(w, act_load(v + 32 * e), o[e] * fo);
        }
        f = l > 0.f ? 1.f / l : 0.f;
    }
    if (a.maps > 1) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < MAXE; e++) o[e] = first[e] - a.lambda * (o[e] * f), ss += o[e] * o[e];
#pragma unroll
        for (int off = 16; off >= 1; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
        f = a.diff_scale / sqrtf(ss / (float)a.vdim + a.eps);
    }
    f *= a.out_scale;
    if (a.gate == GATE_HEAD) f *= sigmoid(act_load(proj + a.g_off + h));
    AT *out = reinterpret_cast<AT *>(a.out) + (size_t)r * a.ldo + a.out_off + h * a.DV + lane;
#pragma unroll
    for (int e = 0; e < MAXE; e++)
        if (e < nv) act_store(out + 32 * e, o[e] * f * (a.gate == GATE_ELEMENT ? sigmoid(act_load(proj + a.g_off + h * a.DV + lane + 32 * e)) : 1.f));
}

// ------------------------------------------------------------------------------------------------
// bf16 on the tensor cores.  A row of a score tile is a (token, head of the group) pair: every query head that shares a key
// head reads the same staged K / V.
// ------------------------------------------------------------------------------------------------
// Factor on a finished row: the head's gate, the branch's scale.
__device__ __forceinline__ float row_factor(const AttnArgs &a, int row, int h) {
    float f = a.out_scale;
    if (a.gate == GATE_HEAD) f *= sigmoid(act_load(reinterpret_cast<const __nv_bfloat16 *>(a.proj) + (size_t)row * a.ldp + a.g_off + h));
    return f;
}
// The gates of the elements from column c of head h on.
__device__ __forceinline__ const __nv_bfloat16 *gate_at(const AttnArgs &a, int row, int h, int c) {
    return reinterpret_cast<const __nv_bfloat16 *>(a.proj) + (size_t)row * a.ldp + a.g_off + h * a.DV + c;
}

// Entries with several tokens (queries are prepared, K / V in the pages).  CTA = 64 rows of one key head: 4 warps x 16 rows for
// each map; tiles of 64 keys through two stages.  The second map's warps hand their rows over in shared memory.
constexpr int kTileKeys = 64;
template <int DK, int DV, int MAPS>
__host__ __device__ constexpr size_t tile_smem() { return (size_t)2 * (MAPS * 64 * (DK + 8) + 2 * kTileKeys * (MAPS * (DK + 8) + DV + 8)); }

template <int DK, int DV, int MAPS>
__global__ void __launch_bounds__(128 * MAPS) attn_tile_kernel(const AttnArgs a, const Seg *__restrict__ segs, const int2 *__restrict__ tiles, int qt, int pdl) {
    constexpr int LK = DK + 8, LV = DV + 8, CK = DK / 8, CV = DV / 8, NT = 128 * MAPS, STAGE = kTileKeys * (MAPS * LK + LV), KW = MAPS * DK;
    extern __shared__ __align__(16) uint8_t attn_smem[];
    __nv_bfloat16 *qs = reinterpret_cast<__nv_bfloat16 *>(attn_smem), *kv_s = qs + MAPS * 64 * LK;  // stages: [K 64 x LK] per map, [V 64 x LV]
    const int tid = threadIdx.x, lane = tid & 31, g = lane >> 2, map = tid / 128, warp = (tid % 128) >> 5;
    const int grp = a.heads / a.kv_heads, kvh = blockIdx.y, r0 = blockIdx.z * 64;
    if (pdl & 2) griddep_launch_dependents();
    const int2 tile = tiles[gridDim.x - 1 - blockIdx.x];  // the last tiles of a prompt see most keys
    const Seg sg = segs[tile.x];
    const int nt = min(qt, sg.T - tile.y), rows = nt * grp, row_base = sg.row0 + tile.y;
    if (r0 >= rows) return;
    const int p0 = sg.pos0 + tile.y, p1 = sg.pos0 + tile.y + (min(rows, r0 + 64) - 1) / grp;
    const __nv_bfloat16 *proj = reinterpret_cast<const __nv_bfloat16 *>(a.proj);
    const __nv_bfloat16 *kv = reinterpret_cast<const __nv_bfloat16 *>(a.kv);
    if (pdl & 1) griddep_wait();
    for (int e = tid; e < MAPS * 64 * CK; e += NT) {
        const int m = e / (64 * CK), r = r0 + e / CK % 64, c = e % CK;
        const bool ok = r < rows;
        const int t = ok ? r / grp : 0, h = kvh * grp + (ok ? r % grp : 0);
        cp_async16(qs + (e / CK) * LK + c * 8, proj + (size_t)(row_base + t) * a.ldp + a.q_off + (h * MAPS + m) * DK + c * 8, ok);
    }
    const int first = first_visible(p0 + r0 / grp, a.chunk) / kBlockTokens * kBlockTokens;
    auto load = [&](int stage, int kb) {
        __nv_bfloat16 *dst = kv_s + (size_t)stage * STAGE;
        for (int e = tid; e < kTileKeys * (MAPS * CK + CV); e += NT) {
            const int j = e / (MAPS * CK + CV), c = e % (MAPS * CK + CV), key = kb + j, m = c / CK;
            const int phys = key <= p1 ? page_of(a, sg.seq, key) : -1;
            const __nv_bfloat16 *src = kv + ((size_t)(phys < 0 ? 0 : phys) * a.kv_heads + kvh) * (kBlockTokens * (KW + DV));
            if (MAPS * CK > c) cp_async16(dst + (m * kTileKeys + j) * LK + c % CK * 8, src + (key % kBlockTokens) * KW + c * 8, phys >= 0);
            else cp_async16(dst + MAPS * kTileKeys * LK + j * LV + (c - MAPS * CK) * 8, src + kBlockTokens * KW + (key % kBlockTokens) * DV + (c - MAPS * CK) * 8, phys >= 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0, first);
    int lo[2], hi[2], rt[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int r = r0 + warp * 16 + g + 8 * e;
        rt[e] = r < rows ? r : -1;
        hi[e] = p0 + (r < rows ? r / grp : r0 / grp);
        lo[e] = first_visible(hi[e], a.chunk);
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    auto qfrag = [&](int kk, uint32_t (&f)[4]) {
        ldmatrix_x4(f, qs + (size_t)(map * 64 + warp * 16 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8);
    };
    const float sl = a.scale * 1.4426950408889634f;
    const int vis_lo = first_visible(p1, a.chunk);
    int it = 0;
    for (int kb = first; kb <= p1; kb += kTileKeys, it++) {
        if (kb + kTileKeys <= p1) {
            load((it + 1) & 1, kb + kTileKeys);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const __nv_bfloat16 *ks = kv_s + (size_t)(it & 1) * STAGE;
        const bool masked = kb + kTileKeys - 1 > p0 + r0 / grp || kb < vis_lo;
        attend_tile<DK, DV, kTileKeys>(qfrag, ks + map * kTileKeys * LK, ks + MAPS * kTileKeys * LK, kb, masked, lo, hi, sl, m, l, o, lane);
        __syncthreads();
    }
    float f[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        f[e] = l[e] > 0.f ? 1.f / l[e] : 0.f;
    }
    if (MAPS == 2) {
        float *other = reinterpret_cast<float *>(kv_s);  // [64][DV + 8]
        const int t2 = 2 * (lane & 3);
        if (map == 1) {
#pragma unroll
            for (int e = 0; e < 2; e++)
#pragma unroll
                for (int n = 0; n < DV / 8; n++)
                    *reinterpret_cast<float2 *>(other + (warp * 16 + g + 8 * e) * LV + n * 8 + t2) = make_float2(o[n][2 * e] * f[e], o[n][2 * e + 1] * f[e]);
        }
        __syncthreads();
        if (map == 1) return;
#pragma unroll
        for (int e = 0; e < 2; e++) {
            float ss = 0.f;
#pragma unroll
            for (int n = 0; n < DV / 8; n++) {
                const float2 b = *reinterpret_cast<const float2 *>(other + (warp * 16 + g + 8 * e) * LV + n * 8 + t2);
                o[n][2 * e] = o[n][2 * e] * f[e] - a.lambda * b.x, o[n][2 * e + 1] = o[n][2 * e + 1] * f[e] - a.lambda * b.y;
                ss += o[n][2 * e] * o[n][2 * e] + o[n][2 * e + 1] * o[n][2 * e + 1];
            }
            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
            f[e] = a.diff_scale / sqrtf(ss / (float)a.vdim + a.eps);
        }
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
        if (rt[e] < 0) continue;
        const int row = row_base + rt[e] / grp, h = kvh * grp + rt[e] % grp, c = 2 * (lane & 3);
        const float fr = f[e] * row_factor(a, row, h);
        __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(a.out) + (size_t)row * a.ldo + a.out_off + h * DV + c;
        const uint32_t *gate = reinterpret_cast<const uint32_t *>(gate_at(a, row, h, c));
#pragma unroll
        for (int n = 0; n < DV / 8; n++) {
            float x = o[n][2 * e] * fr, y = o[n][2 * e + 1] * fr;
            if (a.gate == GATE_ELEMENT) {
                const uint32_t u = gate[n * 4];
                const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&u));
                x *= 1.f / (1.f + __expf(-z.x)), y *= 1.f / (1.f + __expf(-z.y));
            }
            *reinterpret_cast<uint32_t *>(out + n * 8) = bf16_pair(x, y);
        }
    }
}

// Entries with one token: a cluster of CTAs per (entry, key head) cuts the visible pages between them, a warp takes every
// fourth page of its CTA through its own copy ring (no block barrier in the loop), and the partial softmax states meet through
// cluster shared memory.  The query rows are the heads of the group times the maps: with two maps a row is zero outside its own
// map's half of the key, so one product scores both.  With one map CTA r of the cluster finishes its share of the head's columns,
// with two a warp somewhere in the cluster finishes a head.  With FUSED the kernel prepares its heads itself, and the CTA that
// owns the last page writes the token's K and V into it first.
template <int DK, int DV>
__host__ __device__ constexpr int single_stages() { return DK + DV <= 256 ? 3 : 2; }
template <int DK, int DV>
__host__ __device__ constexpr size_t single_ring() {
    const size_t ring = (size_t)4 * single_stages<DK, DV>() * 16 * (DK + DV + 16) * 2, part = sizeof(float) * 4 * 16 * (DV + 4);
    return ring > part ? ring : part;  // the warps' partial states take the ring's place
}
template <int DK, int DV>
__host__ __device__ constexpr size_t single_smem() {
    return single_ring<DK, DV>() + sizeof(float) * 16 * (DV + 4) + (size_t)16 * (DK + 8) * 2;  // the CTA's merged state and the query rows are their own
}

template <int DK, int DV>  // DK: of all maps together
__global__ void __launch_bounds__(128) attn_single_kernel(const AttnArgs a, const Seg *__restrict__ segs, const int *__restrict__ singles, int row_blocks,
                                                          int fused, int pdl) {
    constexpr int LK = DK + 8, LV = DV + 8, CK = DK / 8, CV = DV / 8, ST = single_stages<DK, DV>(), PW = DV + 4, PAGE = 16 * (LK + LV);
    extern __shared__ __align__(16) uint8_t attn_smem[];
    __nv_bfloat16 *ring = reinterpret_cast<__nv_bfloat16 *>(attn_smem);                      // [4 warps][ST][K 16 x LK | V 16 x LV]
    float *part = reinterpret_cast<float *>(attn_smem);                                      // [4 warps][16][m, l, -, -, o[DV]], after the loop
    float *merged = reinterpret_cast<float *>(attn_smem + single_ring<DK, DV>());            // [16][m, l, -, -, o[DV]] of this CTA
    __nv_bfloat16 *qs = reinterpret_cast<__nv_bfloat16 *>(merged + 16 * PW);                 // [16][LK]
    __shared__ float bufs[128 * 8];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = 2 * (lane & 3);
    const int nsplit = gridDim.x, split = blockIdx.x, maps = a.maps, hpb = 16 / maps, dk = DK / maps;
    const int rb = blockIdx.y % row_blocks, kvh = blockIdx.y / row_blocks, grp = a.heads / a.kv_heads, h0 = kvh * grp + rb * hpb, nh = min(hpb, grp - rb * hpb);
    if (pdl & 2) griddep_launch_dependents();
    const Seg sg = segs[singles[blockIdx.z]];
    const int p = sg.pos0, row = sg.row0, first = first_visible(p, a.chunk), lo_page = first / kBlockTokens, n_pages = p / kBlockTokens - lo_page + 1;
    const int pg0 = lo_page + split * n_pages / nsplit, pg1 = lo_page + (split + 1) * n_pages / nsplit;
    const __nv_bfloat16 *proj = reinterpret_cast<const __nv_bfloat16 *>(a.proj) + (size_t)row * a.ldp;
    __nv_bfloat16 *kv = reinterpret_cast<__nv_bfloat16 *>(a.kv);
    for (int e = tid; e < 16 * LK / 8; e += 128) reinterpret_cast<uint4 *>(qs)[e] = make_uint4(0, 0, 0, 0);
    if (pdl & 1) griddep_wait();
    __syncthreads();
    {
        // heads of the group, then (with the last page) the key's maps
        const int lanes = head_lanes(dk), piece = tid & (lanes - 1), slots = 128 / lanes, nq = nh * maps;
        const bool append = fused && split == nsplit - 1;
        const int phys = append ? page_of(a, sg.seq, p) : -1, total = nq + (phys >= 0 ? maps : 0);
        __nv_bfloat16 *page = kv + ((size_t)(phys < 0 ? 0 : phys) * a.kv_heads + kvh) * (16 * (DK + DV));
        for (int v0 = 0; v0 < total; v0 += slots) {
            const int v = v0 + tid / lanes;
            const bool load = v < total && piece * 8 < dk, key = v >= nq;
            float x[8];
            if (load) load8(proj + (key ? a.k_off + (kvh * maps + v - nq) * dk : a.q_off + (h0 * maps + v) * dk) + piece * 8, x);
            else {
#pragma unroll
                for (int e = 0; e < 8; e++) x[e] = 0.f;
            }
            if (fused && a.prepared())
                prepare_head(x, piece, lanes, a.dim, key ? a.k_norm : a.q_norm, a.eps, a.cs + (size_t)row * a.half, a.half, a.interleaved, bufs + (tid - piece) * 8);
            if (!load) continue;
            if (key) store8(page + (size_t)(p % kBlockTokens) * DK + (v - nq) * dk + piece * 8, x);
            else store8(qs + ((v % maps) * hpb + v / maps) * LK + (v % maps) * dk + piece * 8, x);
        }
        if (phys >= 0)
            for (int c = tid; c < CV; c += 128)
                *reinterpret_cast<uint4 *>(page + 16 * DK + (size_t)(p % kBlockTokens) * DV + c * 8) = *reinterpret_cast<const uint4 *>(proj + a.v_off + kvh * DV + c * 8);
        __syncthreads();  // the copies below read what this CTA has just written
    }
    __nv_bfloat16 *mine = ring + (size_t)warp * ST * PAGE;
    // physical blocks of this warp's next 32 pages, a page per lane: one trip to the table instead of one per page
    int blocks = -1;
    auto lookup = [&](int i) {
        const int pg = pg0 + warp + 4 * (i + lane);
        blocks = pg < pg1 ? page_of(a, sg.seq, pg * kBlockTokens) : -1;
    };
    auto load = [&](int i) {  // the i-th page of this warp
        const int pg = pg0 + warp + 4 * i;
        if ((i & 31) == 0) lookup(i);
        const int phys = __shfl_sync(0xffffffffu, blocks, i & 31);
        if (pg < pg1) {
            const __nv_bfloat16 *src = kv + ((size_t)(phys < 0 ? 0 : phys) * a.kv_heads + kvh) * (16 * (DK + DV));
            __nv_bfloat16 *dst = mine + (size_t)(i % ST) * PAGE;
            const int live = phys < 0 ? 0 : p + 1 - pg * kBlockTokens;  // rows of the page that hold tokens
            for (int e = lane; e < 16 * CK; e += 32) cp_async16(dst + e / CK * LK + e % CK * 8, src + e * 8, e / CK < live);
            for (int e = lane; e < 16 * CV; e += 32) cp_async16(dst + 16 * LK + e / CV * LV + e % CV * 8, src + 16 * DK + e * 8, e / CV < live);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int i = 0; i < ST - 1; i++) load(i);
    uint32_t q[DK / 16][4];
#pragma unroll
    for (int kk = 0; kk < DK / 16; kk++) ldmatrix_x4(q[kk], qs + (size_t)(lane & 15) * LK + kk * 16 + (lane >> 4) * 8);
    auto qfrag = [&](int kk, uint32_t (&f)[4]) { f[0] = q[kk][0], f[1] = q[kk][1], f[2] = q[kk][2], f[3] = q[kk][3]; };
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    const int lo[2] = {first, first}, hi[2] = {p, p};
    const float sl = a.scale * 1.4426950408889634f;
    for (int i = 0; pg0 + warp + 4 * i < pg1; i++) {
        asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");
        __syncwarp();
        const __nv_bfloat16 *ks = mine + (size_t)(i % ST) * PAGE;
        const int kb = (pg0 + warp + 4 * i) * kBlockTokens;
        attend_tile<DK, DV, 16>(qfrag, ks, ks + 16 * LK, kb, kb < first || kb + 15 > p, lo, hi, sl, m, l, o, lane);
        __syncwarp();
        load(i + ST - 1);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // every warp is done with its ring
#pragma unroll
    for (int e = 0; e < 2; e++) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        float *w = part + ((size_t)warp * 16 + g + 8 * e) * PW;
        if ((lane & 3) == 0) w[0] = m[e], w[1] = l[e];
#pragma unroll
        for (int n = 0; n < DV / 8; n++) *reinterpret_cast<float2 *>(w + 4 + n * 8 + t2) = make_float2(o[n][2 * e], o[n][2 * e + 1]);
    }
    __syncthreads();
    const int rows = maps == 1 ? nh : hpb + nh;  // with two maps the second one's rows start at hpb
    for (int e = tid; e < rows * DV; e += 128) {
        const int r = e / DV, c = e % DV;
        float mx = -INFINITY, sum = 0.f, acc = 0.f;
#pragma unroll
        for (int w = 0; w < 4; w++) mx = fmaxf(mx, part[(w * 16 + r) * PW]);
#pragma unroll
        for (int w = 0; w < 4; w++) {
            const float *q4 = part + (w * 16 + r) * PW;
            const float f = q4[0] == -INFINITY ? 0.f : fast_exp2(q4[0] - mx);
            sum += f * q4[1], acc += f * q4[4 + c];
        }
        merged[r * PW + 4 + c] = acc;
        if (c == 0) merged[r * PW] = mx, merged[r * PW + 1] = sum;
    }
    if (nsplit > 1) cluster_sync();
    else __syncthreads();
    __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(a.out) + (size_t)row * a.ldo + a.out_off + (size_t)h0 * DV;
    if (maps == 1) {
        const int c0 = split * DV / nsplit, cn = (split + 1) * DV / nsplit - c0;
        for (int e = tid; e < nh * cn; e += 128) {
            const int r = e / cn, c = c0 + e % cn;
            float mx = -INFINITY, sum = 0.f, acc = 0.f;
            if (nsplit == 1) {
                sum = merged[r * PW + 1], acc = merged[r * PW + 4 + c];
            } else {
                for (int s = 0; s < nsplit; s++) mx = fmaxf(mx, ld_cluster_f32(merged + r * PW, (uint32_t)s));
                for (int s = 0; s < nsplit; s++) {
                    const float ms = ld_cluster_f32(merged + r * PW, (uint32_t)s), f = ms == -INFINITY ? 0.f : fast_exp2(ms - mx);
                    sum += f * ld_cluster_f32(merged + r * PW + 1, (uint32_t)s), acc += f * ld_cluster_f32(merged + r * PW + 4 + c, (uint32_t)s);
                }
            }
            float v = acc * (sum > 0.f ? 1.f / sum : 0.f) * row_factor(a, row, h0 + r);
            if (a.gate == GATE_ELEMENT) v *= sigmoid(act_load(gate_at(a, row, h0 + r, c)));
            out[(size_t)r * DV + c] = __float2bfloat16(v);
        }
    } else {
        constexpr int NC = (DV + 127) / 128;  // groups of four columns per lane
        for (int r = split + nsplit * warp; r < nh; r += 4 * nsplit) {
            float4 x[NC];
            float ss = 0.f;
            for (int map = 0; map < 2; map++) {
                const float *at = merged + (map * hpb + r) * PW;
                float mx = -INFINITY, sum = 0.f;
                float4 acc[NC];
#pragma unroll
                for (int n = 0; n < NC; n++) acc[n] = make_float4(0.f, 0.f, 0.f, 0.f);
                for (int s = 0; s < nsplit; s++) mx = fmaxf(mx, ld_cluster_f32(at, (uint32_t)s));
                for (int s = 0; s < nsplit; s++) {
                    const float ms = ld_cluster_f32(at, (uint32_t)s), f = ms == -INFINITY ? 0.f : fast_exp2(ms - mx);
                    sum += f * ld_cluster_f32(at + 1, (uint32_t)s);
#pragma unroll
                    for (int n = 0; n < NC; n++)
                        if (lane * 4 + n * 128 < DV) {
                            const float4 y = ld_cluster_f32x4(at + 4 + lane * 4 + n * 128, (uint32_t)s);
                            acc[n].x += f * y.x, acc[n].y += f * y.y, acc[n].z += f * y.z, acc[n].w += f * y.w;
                        }
                }
                const float f = (sum > 0.f ? 1.f / sum : 0.f) * (map ? -a.lambda : 1.f);
#pragma unroll
                for (int n = 0; n < NC; n++) {
                    if (map == 0) x[n] = make_float4(acc[n].x * f, acc[n].y * f, acc[n].z * f, acc[n].w * f);
                    else x[n].x += acc[n].x * f, x[n].y += acc[n].y * f, x[n].z += acc[n].z * f, x[n].w += acc[n].w * f;
                    if (map == 1) ss += x[n].x * x[n].x + x[n].y * x[n].y + x[n].z * x[n].z + x[n].w * x[n].w;
                }
            }
#pragma unroll
            for (int off = 16; off >= 1; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
            const float f = a.diff_scale / sqrtf(ss / (float)a.vdim + a.eps) * row_factor(a, row, h0 + r);
#pragma unroll
            for (int n = 0; n < NC; n++) {
                const int c = lane * 4 + n * 128;
                if (c >= DV) continue;
                float v[4] = {x[n].x * f, x[n].y * f, x[n].z * f, x[n].w * f};
                if (a.gate == GATE_ELEMENT)
#pragma unroll
                    for (int e = 0; e < 4; e++) v[e] *= sigmoid(act_load(gate_at(a, row, h0 + r, c + e)));
                *reinterpret_cast<uint2 *>(out + (size_t)r * DV + c) = make_uint2(bf16_pair(v[0], v[1]), bf16_pair(v[2], v[3]));
            }
        }
    }
    if (nsplit > 1) cluster_sync();  // nobody leaves while its shared memory is being read
}

// What the kernels are built for.  With two maps DK is the size of one.
struct HeadSizes {
    int maps, DK, DV;
};
constexpr HeadSizes kHeadSizes[] = {{1, 32, 32},  {1, 64, 32},  {1, 64, 64},  {1, 96, 96},  {1, 128, 64}, {1, 128, 128}, {1, 192, 192}, {1, 256, 256},
                                    {2, 32, 32},  {2, 32, 64},  {2, 64, 64},  {2, 64, 96},  {2, 64, 128}, {2, 96, 192},  {2, 128, 128}, {2, 128, 256}};

bool attn_padded_head(int dim, int vdim, int maps, int *DK, int *DV) {
    int best = 0;
    for (const HeadSizes &s : kHeadSizes)
        if (s.maps == maps && dim > 0 && vdim > 0 && dim <= s.DK && vdim <= s.DV && (!best || s.DK + s.DV < best)) best = s.DK + s.DV, *DK = s.DK, *DV = s.DV;
    return best > 0;
}
int attn_query_tile(int heads, int kv_heads) { return std::max(1, 64 / (heads / kv_heads)); }

static long long prep_blocks(const AttnArgs &a, int rows) {
    const long long vectors = (long long)rows * ((a.prepared() ? a.heads * a.maps : 0) + a.kv_heads * (a.maps + 1));
    return (vectors * head_lanes(a.DK) + 255) / 256;
}

template <class AT>
static int32_t rows_attention(const StepDesc &d, const AttnArgs &a, cudaStream_t st) {
    attn_prep_kernel<AT><<<(unsigned)prep_blocks(a, d.rows), 256, 0, st>>>(a, d.seq, d.pos, d.rows, 0);
    attn_rows_kernel<AT><<<(unsigned)((d.rows * (long long)a.heads + 7) / 8), 256, 0, st>>>(a, d.seq, d.pos, d.rows);
    JGPT_CUDA_TRY(cudaGetLastError());
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

template <int MAPS, int DK, int DV>
static int32_t tensor_attention(const StepDesc &d, const AttnArgs &a, int pdl, cudaStream_t st) {
    constexpr int KW = MAPS * DK;
    const int grp = a.heads / a.kv_heads;
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[2];
    cfg.stream = st, cfg.attrs = attr;
    auto early = [&](int n) {
        if (!(pdl & 1)) return n;
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        return n + 1;
    };
    if (d.n_tiles) {
        cfg.gridDim = dim3((unsigned)prep_blocks(a, d.rows)), cfg.blockDim = dim3(256), cfg.dynamicSmemBytes = 0, cfg.numAttrs = (unsigned)early(0);
        JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, attn_prep_kernel<__nv_bfloat16>, a, d.seq, d.pos, d.rows, pdl));
        static thread_local int set_for = -1;
        if (int32_t rc = opt_in(attn_tile_kernel<DK, DV, MAPS>, tile_smem<DK, DV, MAPS>(), set_for)) return rc;
        cfg.gridDim = dim3((unsigned)d.n_tiles, (unsigned)a.kv_heads, (unsigned)((d.qt * grp + 63) / 64)), cfg.blockDim = dim3(128 * MAPS);
        cfg.dynamicSmemBytes = tile_smem<DK, DV, MAPS>(), cfg.numAttrs = (unsigned)early(0);
        JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, attn_tile_kernel<DK, DV, MAPS>, a, d.segs, d.tiles, d.qt, pdl));
    }
    if (d.n_singles) {
        static thread_local int set_for = -1;
        if (int32_t rc = opt_in(attn_single_kernel<KW, DV>, single_smem<KW, DV>(), set_for)) return rc;
        const int row_blocks = (grp * MAPS + 15) / 16, ctas = d.n_singles * a.kv_heads * row_blocks;
        const int keys = a.chunk > 0 ? std::min(a.chunk, d.max_len) : d.max_len, pages = keys / kBlockTokens + 1;
        int split = 1;  // every warp keeps two pages, the grid stays around two CTAs per SM
        while (split < 8 && ctas * split * 2 <= 2 * a.sm_count && pages >= split * 2 * 8) split *= 2;
        int na = early(0);
        if (split > 1) {
            attr[na].id = cudaLaunchAttributeClusterDimension;
            attr[na].val.clusterDim.x = (unsigned)split, attr[na].val.clusterDim.y = 1, attr[na].val.clusterDim.z = 1;
            na++;
        }
        cfg.gridDim = dim3((unsigned)split, (unsigned)(a.kv_heads * row_blocks), (unsigned)d.n_singles), cfg.blockDim = dim3(128);
        cfg.dynamicSmemBytes = single_smem<KW, DV>(), cfg.numAttrs = (unsigned)na;
        JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, attn_single_kernel<KW, DV>, a, d.segs, d.singles, row_blocks, d.n_tiles ? 0 : 1, pdl));
    }
    return JGPT_OK;
}

template <int I = 0>
static int32_t pick_attention(const StepDesc &d, const AttnArgs &a, int pdl, cudaStream_t st) {
    if constexpr (I < (int)(sizeof(kHeadSizes) / sizeof(kHeadSizes[0]))) {
        constexpr HeadSizes s = kHeadSizes[I];
        if (a.maps == s.maps && a.DK == s.DK && a.DV == s.DV) return tensor_attention<s.maps, s.DK, s.DV>(d, a, pdl, st);
        return pick_attention<I + 1>(d, a, pdl, st);
    } else {
        return fail(JGPT_ERR_UNSUPPORTED, "head sizes %d / %d", a.DK, a.DV);
    }
}

int32_t launch_attention(bool f32, const StepDesc &d, const AttnArgs &a, int pdl, cudaStream_t st) {
    return f32 ? rows_attention<float>(d, a, st) : pick_attention(d, a, pdl, st);
}

}  // namespace mix
}  // namespace jgpt
