// Paged attention of the layered decoder: query heads in groups that share a key head, head sizes up to 256 (padded to a
// multiple of 32), a visibility rule by chunks of positions, an optional output gate per head.
//
//   attn_append_kernel   rows of K and V into the pages (in the cache's type; no rotation)
//   attn_rows_kernel     one warp per (row, head), fp32: the exact mode
//   attn_tile_kernel     portions of prompts, bf16 tensor cores
//   attn_single_kernel   single tokens, bf16 tensor cores over a split sequence
#include "mixers.cuh"

#include <algorithm>

#include "attn_mma.cuh"

namespace jgpt {
namespace mix {

__host__ __device__ __forceinline__ int first_visible(int pos, int chunk) { return chunk > 0 ? pos / chunk * chunk : 0; }

// One thread moves 16 bytes of one (row, key head) of K and of V.
template <class AT>
__global__ void __launch_bounds__(256) attn_append_kernel(const AttnArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int rows,
                                                          int pdl) {
    constexpr int E = 16 / sizeof(AT);
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    const int cpr = a.D / E;
    const long long gid = (long long)blockIdx.x * 256 + threadIdx.x;
    if (gid >= (long long)rows * a.kv_heads * cpr) return;
    const int c = (int)(gid % cpr), g = (int)(gid / cpr % a.kv_heads), r = (int)(gid / ((long long)cpr * a.kv_heads));
    const int p = pos[r], phys = page_of(a, seq[r], p);
    if (phys < 0) return;
    const AT *src = reinterpret_cast<const AT *>(a.proj) + (size_t)r * a.ldp + g * a.D + c * E;
    AT *dst = reinterpret_cast<AT *>(a.kv) + ((size_t)phys * a.kv_heads + g) * (2 * kBlockTokens * a.D) + (size_t)(p % kBlockTokens) * a.D + c * E;
    *reinterpret_cast<uint4 *>(dst) = *reinterpret_cast<const uint4 *>(src + a.k_off);
    *reinterpret_cast<uint4 *>(dst + kBlockTokens * a.D) = *reinterpret_cast<const uint4 *>(src + a.v_off);
}

// One warp per (row, query head): lane l holds elements l, l + 32, ... of q and of the output.
template <class AT>
__global__ void __launch_bounds__(256) attn_rows_kernel(const AttnArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int rows) {
    constexpr int MAXE = 8;
    const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= rows * a.heads) return;
    const int r = item / a.heads, h = item % a.heads, g = h / (a.heads / a.kv_heads), ne = a.D / 32;
    const AT *proj = reinterpret_cast<const AT *>(a.proj) + (size_t)r * a.ldp;
    float q[MAXE], o[MAXE];
#pragma unroll
    for (int e = 0; e < MAXE; e++) q[e] = e < ne ? act_load(proj + a.q_off + h * a.D + lane + 32 * e) * a.scale : 0.f, o[e] = 0.f;
    float m = -INFINITY, l = 0.f;
    const int p = pos[r], s = seq[r];
    for (int j = first_visible(p, a.chunk); j <= p; j++) {
        const int phys = page_of(a, s, j);
        if (phys < 0) break;
        const AT *k = reinterpret_cast<const AT *>(a.kv) + ((size_t)phys * a.kv_heads + g) * (2 * kBlockTokens * a.D) +
                      (size_t)(j % kBlockTokens) * a.D + lane;
        float d = 0.f;
#pragma unroll
        for (int e = 0; e < MAXE; e++)
            if (e < ne) d = fmaf(q[e], act_load(k + 32 * e), d);
#pragma unroll
        for (int off = 16; off >= 1; off >>= 1) d += __shfl_xor_sync(0xffffffffu, d, off);
        const float mn = fmaxf(m, d), f = expf(m - mn), w = expf(d - mn);
        m = mn, l = l * f + w;
#pragma unroll
        for (int e = 0; e < MAXE; e++)
            if (e < ne) o[e] = fmaf(w, act_load(k + kBlockTokens * a.D + 32 * e), o[e] * f);
    }
    float f = (l > 0.f ? 1.f / l : 0.f) * a.out_scale;
    if (a.g_off >= 0) f *= 1.f / (1.f + expf(-act_load(proj + a.g_off + h)));
    AT *out = reinterpret_cast<AT *>(a.out) + (size_t)r * a.ldo + a.out_off + h * a.D + lane;
#pragma unroll
    for (int e = 0; e < MAXE; e++)
        if (e < ne) act_store(out + 32 * e, o[e] * f);
}

// ------------------------------------------------------------------------------------------------
// bf16 on the tensor cores.  A row of a score tile is a (token, head of the group) pair: every query head that shares a key
// head reads the same staged K / V.
// ------------------------------------------------------------------------------------------------
// Factor on a finished row: 1 / sum of weights, the output gate, the branch's scale.
__device__ __forceinline__ float row_factor(const AttnArgs &a, int row, int h, float l) {
    float f = (l > 0.f ? 1.f / l : 0.f) * a.out_scale;
    if (a.g_off >= 0) f *= 1.f / (1.f + expf(-act_load(reinterpret_cast<const __nv_bfloat16 *>(a.proj) + (size_t)row * a.ldp + a.g_off + h)));
    return f;
}

// Entries with several tokens (K / V are in the pages already).  CTA = 64 rows of one key head: 4 warps x 16 rows; tiles of
// 64 keys through two stages.
constexpr int kTileKeys = 64;
template <int D>
__host__ __device__ constexpr size_t tile_smem() { return (size_t)(64 + 4 * kTileKeys) * (D + 8) * 2; }

template <int D>
__global__ void __launch_bounds__(128) attn_tile_kernel(const AttnArgs a, const Seg *__restrict__ segs, const int2 *__restrict__ tiles, int qt, int pdl) {
    constexpr int LD = D + 8, CH = D / 8;
    extern __shared__ __align__(16) uint8_t attn_smem[];
    __nv_bfloat16 *qs = reinterpret_cast<__nv_bfloat16 *>(attn_smem), *kv_s = qs + 64 * LD;  // stages: [K 64 x LD | V 64 x LD]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2;
    const int grp = a.heads / a.kv_heads, kvh = blockIdx.y, r0 = blockIdx.z * 64;
    if (pdl & 2) griddep_launch_dependents();
    const int2 tile = tiles[blockIdx.x];
    const Seg sg = segs[tile.x];
    const int nt = min(qt, sg.T - tile.y), rows = nt * grp, row_base = sg.row0 + tile.y;
    if (r0 >= rows) return;
    const int p0 = sg.pos0 + tile.y, p1 = p0 + nt - 1;
    const __nv_bfloat16 *proj = reinterpret_cast<const __nv_bfloat16 *>(a.proj);
    const __nv_bfloat16 *kv = reinterpret_cast<const __nv_bfloat16 *>(a.kv);
    if (pdl & 1) griddep_wait();
    for (int e = tid; e < 64 * CH; e += 128) {
        const int r = r0 + e / CH, c = e % CH;
        const bool ok = r < rows;
        const int t = ok ? r / grp : 0, h = kvh * grp + (ok ? r % grp : 0);
        cp_async16(qs + (e / CH) * LD + c * 8, proj + (size_t)(row_base + t) * a.ldp + a.q_off + h * D + c * 8, ok);
    }
    const int first = first_visible(p0, a.chunk) / kBlockTokens * kBlockTokens;
    auto load = [&](int stage, int kb) {
        __nv_bfloat16 *dst = kv_s + (size_t)stage * 2 * kTileKeys * LD;
        for (int e = tid; e < kTileKeys * CH; e += 128) {
            const int j = e / CH, c = e % CH, key = kb + j;
            int phys = key <= p1 ? page_of(a, sg.seq, key) : -1;
            const __nv_bfloat16 *src = kv + ((size_t)(phys < 0 ? 0 : phys) * a.kv_heads + kvh) * (2 * kBlockTokens * D) + (key % kBlockTokens) * D + c * 8;
            cp_async16(dst + j * LD + c * 8, src, phys >= 0);
            cp_async16(dst + (kTileKeys + j) * LD + c * 8, src + kBlockTokens * D, phys >= 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0, first);
    int lo[2], hi[2], rt[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int r = r0 + warp * 16 + g + 8 * e;
        rt[e] = r < rows ? r : -1;
        hi[e] = p0 + (r < rows ? r / grp : 0);
        lo[e] = first_visible(hi[e], a.chunk);
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[D / 8][4];
#pragma unroll
    for (int n = 0; n < D / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    auto qfrag = [&](int kk, uint32_t (&f)[4]) {
        ldmatrix_x4(f, qs + (size_t)(warp * 16 + (lane & 15)) * LD + kk * 16 + (lane >> 4) * 8);
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
        const __nv_bfloat16 *ks = kv_s + (size_t)(it & 1) * 2 * kTileKeys * LD;
        const bool masked = kb + kTileKeys - 1 > p0 || kb < vis_lo;
        attend_tile<D, D, kTileKeys>(qfrag, ks, ks + kTileKeys * LD, kb, masked, lo, hi, sl, m, l, o, lane);
        __syncthreads();
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        if (rt[e] < 0) continue;
        const int row = row_base + rt[e] / grp, h = kvh * grp + rt[e] % grp;
        const float f = row_factor(a, row, h, l[e]);
        __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(a.out) + (size_t)row * a.ldo + a.out_off + h * D + 2 * (lane & 3);
#pragma unroll
        for (int n = 0; n < D / 8; n++) *reinterpret_cast<uint32_t *>(out + n * 8) = bf16_pair(o[n][2 * e] * f, o[n][2 * e + 1] * f);
    }
}

// Entries with one token: a cluster of CTAs per (entry, key head) cuts the visible pages between them, a warp takes every
// fourth page of its CTA through its own copy ring (no block barrier in the loop), and the partial softmax states meet through
// cluster shared memory: CTA r of the cluster finishes its share of the head's columns.  With APPEND the CTA that owns the last page
// writes the token's K and V into it first.
template <int D>
__host__ __device__ constexpr int single_stages() { return D <= 128 ? 3 : 2; }
template <int D>
__host__ __device__ constexpr size_t single_smem() {
    const size_t ring = (size_t)4 * single_stages<D>() * 32 * (D + 8) * 2, part = sizeof(float) * 16 * (D + 2);
    return ring + part;  // the warps' partial states take the ring's place; the CTA's merged state is its own
}

template <int D>
__global__ void __launch_bounds__(128) attn_single_kernel(const AttnArgs a, const Seg *__restrict__ segs, const int *__restrict__ singles, int row_blocks,
                                                          int append, int pdl) {
    constexpr int LD = D + 8, CH = D / 8, ST = single_stages<D>(), PW = D + 2;
    extern __shared__ __align__(16) uint8_t attn_smem[];
    __nv_bfloat16 *ring = reinterpret_cast<__nv_bfloat16 *>(attn_smem);                              // [4 warps][ST][K 16 x LD | V 16 x LD]
    float *part = reinterpret_cast<float *>(attn_smem);                                              // [4 warps][16][m, l, o[D]], after the loop
    float *merged = reinterpret_cast<float *>(attn_smem + (size_t)4 * ST * 32 * LD * 2);             // [16][m, l, o[D]] of this CTA
    static_assert((size_t)4 * ST * 32 * LD * 2 >= sizeof(float) * 4 * 16 * PW, "partial states must fit the ring");
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = 2 * (lane & 3);
    const int nsplit = gridDim.x, split = blockIdx.x;
    const int rb = blockIdx.y % row_blocks, kvh = blockIdx.y / row_blocks, grp = a.heads / a.kv_heads, r0 = rb * 16;
    if (pdl & 2) griddep_launch_dependents();
    const Seg sg = segs[singles[blockIdx.z]];
    const int p = sg.pos0, row = sg.row0, first = first_visible(p, a.chunk), lo_page = first / kBlockTokens, n_pages = p / kBlockTokens - lo_page + 1;
    const int pg0 = lo_page + split * n_pages / nsplit, pg1 = lo_page + (split + 1) * n_pages / nsplit;
    const __nv_bfloat16 *proj = reinterpret_cast<const __nv_bfloat16 *>(a.proj) + (size_t)row * a.ldp;
    __nv_bfloat16 *kv = reinterpret_cast<__nv_bfloat16 *>(a.kv);
    if (pdl & 1) griddep_wait();
    if (append && split == nsplit - 1) {
        const int phys = page_of(a, sg.seq, p);
        if (phys >= 0) {
            __nv_bfloat16 *dst = kv + ((size_t)phys * a.kv_heads + kvh) * (2 * kBlockTokens * D) + (size_t)(p % kBlockTokens) * D;
            for (int c = tid; c < 2 * CH; c += 128) {
                const int which = c / CH, cc = (c % CH) * 8;
                *reinterpret_cast<uint4 *>(dst + which * kBlockTokens * D + cc) =
                    *reinterpret_cast<const uint4 *>(proj + (which ? a.v_off : a.k_off) + kvh * D + cc);
            }
        }
        __syncthreads();  // the copies below read what this CTA has just written
    }
    __nv_bfloat16 *mine = ring + (size_t)warp * ST * 32 * LD;
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
            const __nv_bfloat16 *src = kv + ((size_t)(phys < 0 ? 0 : phys) * a.kv_heads + kvh) * (2 * kBlockTokens * D);
            __nv_bfloat16 *dst = mine + (size_t)(i % ST) * 32 * LD;
            for (int e = lane; e < 32 * CH; e += 32) {
                const int r = e / CH, c = e % CH;
                cp_async16(dst + r * LD + c * 8, src + r * D + c * 8, phys >= 0 && pg * kBlockTokens + (r & 15) <= p);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int i = 0; i < ST - 1; i++) load(i);
    uint32_t q[D / 16][4];
    {
        const bool ok[2] = {r0 + g < grp, r0 + g + 8 < grp};
        const __nv_bfloat16 *qa = proj + a.q_off + (size_t)(kvh * grp + r0) * D + t2;
#pragma unroll
        for (int kk = 0; kk < D / 16; kk++)
#pragma unroll
            for (int e = 0; e < 4; e++)
                q[kk][e] = ok[e & 1] ? *reinterpret_cast<const uint32_t *>(qa + (size_t)(g + 8 * (e & 1)) * D + kk * 16 + (e >> 1) * 8) : 0u;
    }
    auto qfrag = [&](int kk, uint32_t (&f)[4]) { f[0] = q[kk][0], f[1] = q[kk][1], f[2] = q[kk][2], f[3] = q[kk][3]; };
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[D / 8][4];
#pragma unroll
    for (int n = 0; n < D / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    const int lo[2] = {first, first}, hi[2] = {p, p};
    const float sl = a.scale * 1.4426950408889634f;
    for (int i = 0; pg0 + warp + 4 * i < pg1; i++) {
        asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");
        __syncwarp();
        const __nv_bfloat16 *ks = mine + (size_t)(i % ST) * 32 * LD;
        const int kb = (pg0 + warp + 4 * i) * kBlockTokens;
        attend_tile<D, D, 16>(qfrag, ks, ks + 16 * LD, kb, kb < first || kb + 15 > p, lo, hi, sl, m, l, o, lane);
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
        for (int n = 0; n < D / 8; n++) *reinterpret_cast<float2 *>(w + 2 + n * 8 + t2) = make_float2(o[n][2 * e], o[n][2 * e + 1]);
    }
    __syncthreads();
    const int rows = min(16, grp - r0);
    for (int e = tid; e < rows * D; e += 128) {
        const int r = e / D, c = e % D;
        float mx = -INFINITY, sum = 0.f, acc = 0.f;
#pragma unroll
        for (int w = 0; w < 4; w++) mx = fmaxf(mx, part[(w * 16 + r) * PW]);
#pragma unroll
        for (int w = 0; w < 4; w++) {
            const float *q4 = part + (w * 16 + r) * PW;
            const float f = q4[0] == -INFINITY ? 0.f : fast_exp2(q4[0] - mx);
            sum += f * q4[1], acc += f * q4[2 + c];
        }
        merged[r * PW + 2 + c] = acc;
        if (c == 0) merged[r * PW] = mx, merged[r * PW + 1] = sum;
    }
    if (nsplit > 1) cluster_sync();
    else __syncthreads();
    __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(a.out) + (size_t)row * a.ldo + a.out_off + (size_t)(kvh * grp + r0) * D;
    const int c0 = split * D / nsplit, cn = (split + 1) * D / nsplit - c0;
    for (int e = tid; e < rows * cn; e += 128) {
        const int r = e / cn, c = c0 + e % cn;
        float mx = -INFINITY, sum = 0.f, acc = 0.f, v;
        if (nsplit == 1) {
            sum = merged[r * PW + 1], acc = merged[r * PW + 2 + c];
        } else {
            for (int s = 0; s < nsplit; s++) mx = fmaxf(mx, ld_cluster_f32(merged + r * PW, (uint32_t)s));
            for (int s = 0; s < nsplit; s++) {
                const float ms = ld_cluster_f32(merged + r * PW, (uint32_t)s), f = ms == -INFINITY ? 0.f : fast_exp2(ms - mx);
                sum += f * ld_cluster_f32(merged + r * PW + 1, (uint32_t)s), acc += f * ld_cluster_f32(merged + r * PW + 2 + c, (uint32_t)s);
            }
        }
        v = acc * row_factor(a, row, kvh * grp + r0 + r, sum);
        out[(size_t)r * D + c] = __float2bfloat16(v);
    }
    if (nsplit > 1) cluster_sync();  // nobody leaves while its shared memory is being read
}

int attn_padded_head(int dim, int vdim) {
    const int d = std::max(dim, vdim);
    for (int p : {32, 64, 96, 128, 192, 256})
        if (d <= p) return dim > 0 && vdim > 0 ? p : 0;
    return 0;
}
int attn_query_tile(int heads, int kv_heads) { return std::max(1, 64 / (heads / kv_heads)); }

template <class AT>
static int32_t rows_attention(const StepDesc &d, const AttnArgs &a, cudaStream_t st) {
    const long long total = (long long)d.rows * a.kv_heads * (a.D / (16 / (int)sizeof(AT)));
    attn_append_kernel<AT><<<(unsigned)((total + 255) / 256), 256, 0, st>>>(a, d.seq, d.pos, d.rows, 0);
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

template <int D>
static int32_t tensor_attention(const StepDesc &d, const AttnArgs &a, int pdl, cudaStream_t st) {
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
        const long long total = (long long)d.rows * a.kv_heads * (D / 8);
        cfg.gridDim = dim3((unsigned)((total + 255) / 256)), cfg.blockDim = dim3(256), cfg.dynamicSmemBytes = 0, cfg.numAttrs = (unsigned)early(0);
        JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, attn_append_kernel<__nv_bfloat16>, a, d.seq, d.pos, d.rows, pdl));
        static thread_local int set_for = -1;
        if (int32_t rc = opt_in(attn_tile_kernel<D>, tile_smem<D>(), set_for)) return rc;
        cfg.gridDim = dim3((unsigned)d.n_tiles, (unsigned)a.kv_heads, (unsigned)((d.qt * grp + 63) / 64)), cfg.blockDim = dim3(128);
        cfg.dynamicSmemBytes = tile_smem<D>(), cfg.numAttrs = (unsigned)early(0);
        JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, attn_tile_kernel<D>, a, d.segs, d.tiles, d.qt, pdl));
    }
    if (d.n_singles) {
        static thread_local int set_for = -1;
        if (int32_t rc = opt_in(attn_single_kernel<D>, single_smem<D>(), set_for)) return rc;
        const int row_blocks = (grp + 15) / 16, ctas = d.n_singles * a.kv_heads * row_blocks;
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
        cfg.dynamicSmemBytes = single_smem<D>(), cfg.numAttrs = (unsigned)na;
        JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, attn_single_kernel<D>, a, d.segs, d.singles, row_blocks, d.n_tiles ? 0 : 1, pdl));
    }
    return JGPT_OK;
}

int32_t launch_attention(bool f32, const StepDesc &d, const AttnArgs &a, int pdl, cudaStream_t st) {
    if (f32) return rows_attention<float>(d, a, st);
    switch (a.D) {
        case 32: return tensor_attention<32>(d, a, pdl, st);
        case 64: return tensor_attention<64>(d, a, pdl, st);
        case 96: return tensor_attention<96>(d, a, pdl, st);
        case 128: return tensor_attention<128>(d, a, pdl, st);
        case 192: return tensor_attention<192>(d, a, pdl, st);
        case 256: return tensor_attention<256>(d, a, pdl, st);
        default: return fail(JGPT_ERR_UNSUPPORTED, "head size %d", a.D);
    }
}

}  // namespace mix
}  // namespace jgpt
