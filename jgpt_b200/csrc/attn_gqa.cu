// Paged attention of the layered decoder: query heads in groups that share a key head, head sizes up to 256 (padded to what
// the kernels are built for), all earlier positions, those of the query's chunk, or a window and the first tokens, optional norms
// and rotation of the heads, sinks, values mixed with another layer's, one or two maps per head (mixers.cuh), an optional output
// gate per head or per element.
//
//   attn_prep_kernel     keys (normed and rotated) and values into the pages; in the exact mode query heads in place
//   attn_rows_kernel     one warp per (row, head), fp32: the exact mode
//   attn_tile_kernel     portions of prompts, bf16 tensor cores; prepares its query heads
//   attn_single_kernel   single tokens, bf16 tensor cores over a split sequence; prepares its query heads, and its key unless
//                        attn_prep_kernel has done so
#include "mixers.cuh"

#include <algorithm>

#include "attn_mma.cuh"

namespace jgpt {
namespace mix {

// First key of the chunk or window of a position; with a window the keys before a.keep are seen as well.
template <bool WINDOW = true>
__host__ __device__ __forceinline__ int first_visible(int pos, const AttnArgs &a) {
    if (WINDOW && a.window > 0) return pos >= a.window ? pos - a.window + 1 : 0;
    return a.chunk > 0 ? pos / a.chunk * a.chunk : 0;
}
// Keys in front of the window that are visited on their own: none, or [0, keep) when the window's first page lies behind them.
__device__ __forceinline__ int kept_apart(int first_page_key, const AttnArgs &a) { return a.keep > 0 && first_page_key >= a.keep ? a.keep : 0; }

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// What happens to a query or key head (map) behind its projection: norm, rotation.
struct HeadPrep {
    const float *w;  // null: no norm
    const float2 *cs;
    int dim, half, interleaved, whole;
    float eps, inv;  // inv: of the whole row
};
// head: which of the row's (its weights, when the whole row has some); inv: 1 / root mean square of the row, when that is what the norm takes
template <bool WHOLE>
__device__ __forceinline__ HeadPrep head_prep(const AttnArgs &a, bool key, int row, int head, float inv) {
    const float *w = key ? a.k_norm : a.q_norm;
    const bool whole = WHOLE && a.whole_rows;
    return HeadPrep{w + (whole ? head * a.DK : 0), a.cs + (size_t)row * a.half, a.dim, a.half, a.interleaved, whole, a.eps, inv};
}
// The head lies in 8-element pieces in `lanes` neighbouring lanes (a power of two; every lane of the warp takes part); src: its
// start in memory.
template <class AT>
__device__ __forceinline__ void prepare_head(float (&x)[8], const AT *src, int piece, int lanes, const HeadPrep &h) {
    const int j0 = piece * 8;
    float inv = 1.f;
    if (h.w) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; e++) ss += x[e] * x[e];
        for (int off = lanes >> 1; off >= 1; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
        inv = h.whole ? h.inv : 1.f / sqrtf(ss / (float)h.dim + h.eps);
#pragma unroll
        for (int e = 0; e < 8; e++) x[e] = j0 + e < h.dim ? x[e] * inv * __ldg(h.w + j0 + e) : 0.f;
    }
    if (!h.half) return;
    if (h.interleaved) {
#pragma unroll
        for (int e = 0; e < 8; e += 2)
            if (j0 + e < 2 * h.half) {
                const float2 t = h.cs[((j0 + e) >> 1)];
                const float u = x[e], v = x[e + 1];
                x[e] = u * t.x - v * t.y, x[e + 1] = v * t.x + u * t.y;
            }
    } else if ((h.half & 7) == 0) {  // the other element of a pair is in the same place of another lane
        const int hp = h.half >> 3, lane = threadIdx.x & 31;
        const bool first = piece < hp, turns = piece < 2 * hp;
        const int other = turns ? (first ? lane + hp : lane - hp) : lane;
#pragma unroll
        for (int e = 0; e < 8; e++) {
            const float y = __shfl_sync(0xffffffffu, x[e], other);
            if (!turns) continue;
            const float2 t = h.cs[(first ? j0 + e : j0 + e - h.half)];
            x[e] = first ? x[e] * t.x - y * t.y : x[e] * t.x + y * t.y;
        }
    } else {
#pragma unroll
        for (int e = 0; e < 8; e++) {
            const int j = j0 + e, p = j < h.half ? j + h.half : j - h.half;
            if (j >= 2 * h.half) continue;
            const float2 t = h.cs[(j < h.half ? j : p)];
            const float y = act_load(src + p) * inv * (h.w ? __ldg(h.w + p) : 1.f);
            x[e] = j < h.half ? x[e] * t.x - y * t.y : x[e] * t.x + y * t.y;
        }
        __syncwarp();  // whoever writes the head back does so after this
    }
}
__host__ __device__ constexpr int head_lanes(int DK) { return DK <= 32 ? 4 : (DK <= 64 ? 8 : (DK <= 128 ? 16 : 32)); }

// 1 / root mean square of all query heads and of all key heads of a row (padding is zero), by all threads of the block.
template <class AT>
__device__ __forceinline__ float2 row_rms(const AT *proj, const AttnArgs &a, float2 *red) {
    float2 ss = make_float2(0.f, 0.f);
    const int nq = a.heads * a.DK, n = nq + a.kv_heads * a.DK;
    for (int c = threadIdx.x * 8; c < n; c += blockDim.x * 8) {
        float x[8], s = 0.f;
        load8(proj + (c < nq ? a.q_off + c : a.k_off + c - nq), x);
#pragma unroll
        for (int e = 0; e < 8; e++) s += x[e] * x[e];
        if (c < nq) ss.x += s;
        else ss.y += s;
    }
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) ss.x += __shfl_xor_sync(0xffffffffu, ss.x, off), ss.y += __shfl_xor_sync(0xffffffffu, ss.y, off);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = make_float2(0.f, 0.f);
    for (int w = 0; w < (int)blockDim.x / 32; w++) ss.x += red[w].x, ss.y += red[w].y;
    return make_float2(1.f / sqrtf(ss.x / (float)(a.heads * a.dim) + a.eps), 1.f / sqrtf(ss.y / (float)(a.kv_heads * a.dim) + a.eps));
}

// Values of a key head from column c on, mixed with another layer's, whose heads may be cut differently.
__device__ __forceinline__ bool values_line_up(const AttnArgs &a, int c) { return !a.v_first || (a.vdim_first == a.vdim && c + 8 <= a.DV_first); }
template <class AT>
__device__ __forceinline__ void load_values(const AttnArgs &a, int row, int g, int c, float (&x)[8]) {  // eight that line up
    load8(reinterpret_cast<const AT *>(a.proj) + (size_t)row * a.ldp + a.v_off + g * a.DV + c, x);
    if (!a.v_first) return;
    float y[8];
    load8(reinterpret_cast<const AT *>(a.v_first) + (size_t)row * a.ld_first + g * a.DV_first + c, y);
#pragma unroll
    for (int e = 0; e < 8; e++) x[e] = fmaf(a.v_share, y[e], (1.f - a.v_share) * x[e]);
}
template <class AT>
__device__ __forceinline__ float load_value(const AttnArgs &a, int row, int g, int c) {
    if (c >= a.vdim) return 0.f;
    const int i = g * a.vdim + c;
    const float x = act_load(reinterpret_cast<const AT *>(a.proj) + (size_t)row * a.ldp + a.v_off + g * a.DV + c);
    return fmaf(a.v_share, act_load(reinterpret_cast<const AT *>(a.v_first) + (size_t)row * a.ld_first + i / a.vdim_first * a.DV_first + i % a.vdim_first), (1.f - a.v_share) * x);
}

// A block (or several, in y) per row: its query maps (with `queries`, in place), key maps and values (into the page), a vector per
// head_lanes(DK) lanes.  WIDE: norms over the whole row, by the one block that has it, and mixed values.
template <class AT, bool WIDE>
__global__ void __launch_bounds__(256, sizeof(AT) == 2 ? (WIDE ? 6 : 8) : 1) attn_prep_kernel(const AttnArgs a, const int *__restrict__ seq, const int *__restrict__ pos, int queries, int pdl) {
    __shared__ float2 red[8];
    if (pdl & 2) griddep_launch_dependents();
    const int lanes = head_lanes(a.DK), nq = queries ? a.heads * a.maps : 0, nk = a.kv_heads * a.maps, nv = nq + nk + a.kv_heads;
    const int r = blockIdx.x, piece = threadIdx.x & (lanes - 1), per = blockDim.x / lanes;
    const int p = pos[r], row = p % kBlockTokens, phys = page_of(a, seq[r], p), kw = a.maps * a.DK;
    if (pdl & 1) griddep_wait();
    AT *proj = reinterpret_cast<AT *>(a.proj) + (size_t)r * a.ldp;
    float2 inv = make_float2(1.f, 1.f);
    if (WIDE && a.whole_rows) {
        inv = row_rms(proj, a, red);
        if (threadIdx.x == 0) a.row_inv[r] = inv;
    }
#pragma unroll 1
    for (int i0 = blockIdx.y * per; i0 < nv; i0 += gridDim.y * per) {
        const int i = i0 + threadIdx.x / lanes;
        const bool query = i < nq, value = i >= nq + nk && i < nv, key = i >= nq && i < nq + nk;
        const int g = key ? (i - nq) / a.maps : (value ? i - nq - nk : 0);
        AT *page = reinterpret_cast<AT *>(a.kv) + ((size_t)max(phys, 0) * a.kv_heads + g) * a.page_head();
        if (value && phys >= 0) {
            AT *dst = page + kBlockTokens * page_row(kw) + row * page_row(a.DV);
#pragma unroll 1
            for (int c = piece; c < a.DV / 8; c += lanes) {
                float x[8];
                if (WIDE && !values_line_up(a, c * 8)) {
#pragma unroll 1
                    for (int e = 0; e < 8; e++) act_store(dst + page_chunk(a.DV, row, c) * 8 + e, load_value<AT>(a, r, g, c * 8 + e));
                    continue;
                }
                if (WIDE) load_values<AT>(a, r, g, c * 8, x);
                else load8(proj + a.v_off + g * a.DV + c * 8, x);
                store8(dst + page_chunk(a.DV, row, c) * 8, x);
            }
        }
        const int head = query ? i : (key ? i - nq : 0);
        const AT *src = proj + (query ? a.q_off : a.k_off) + head * a.DK;
        float x[8];
        const bool load = (query || key) && piece * 8 < a.DK;
        if (load) load8(src + piece * 8, x);
        else {
#pragma unroll
            for (int e = 0; e < 8; e++) x[e] = 0.f;
        }
        if (a.prepared()) prepare_head(x, src, piece, lanes, head_prep<WIDE>(a, !query, r, head, query ? inv.x : inv.y));
        if (load && query) store8(proj + a.q_off + i * a.DK + piece * 8, x);
        else if (load && phys >= 0) store8(page + row * page_row(kw) + page_chunk(kw, row, (i - nq) % a.maps * (a.DK / 8) + piece) * 8, x);
        if (!WIDE) break;
    }
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
        const int seen = first_visible(p, a);
        for (int j = min(a.keep, seen) > 0 ? 0 : seen; j <= p; j++) {
            if (j == min(a.keep, seen)) j = seen;
            const int phys = page_of(a, s, j);
            if (phys < 0) break;
            const int row = j % kBlockTokens;
            const AT *k = reinterpret_cast<const AT *>(a.kv) + ((size_t)phys * a.kv_heads + g) * a.page_head() + row * page_row(kw);
            const AT *v = k + kBlockTokens * page_row(kw) + row * (page_row(a.DV) - page_row(kw));
            auto at = [&](int D, int e) { return page_chunk(D, row, e >> 3) * 8 + (e & 7); };
            float d = 0.f;
#pragma unroll
            for (int e = 0; e < MAXE; e++)
                if (e < nk) d = fmaf(q[e], act_load(k + at(kw, map * a.DK + lane + 32 * e)), d);
#pragma unroll
            for (int off = 16; off >= 1; off >>= 1) d += __shfl_xor_sync(0xffffffffu, d, off);
            const float mn = fmaxf(m, d), fo = expf(m - mn), w = expf(d - mn);
            m = mn, l = l * fo + w;
#pragma unroll
            for (int e = 0; e < MAXE; e++)
                if (e < nv) o[e] = fmaf(w, act_load(v + at(a.DV, lane + 32 * e)), o[e] * fo);
        }
        if (a.sink) {
            const float mn = fmaxf(m, a.sink[h]), fo = expf(m - mn);
            l = l * fo + expf(a.sink[h] - mn);
#pragma unroll
            for (int e = 0; e < MAXE; e++) o[e] *= fo;
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

// Pages of a key head: 16 rows of K (all maps), 16 of V.
template <int KW, int DV>
struct Page {
    static constexpr int LK = page_row(KW), LV = page_row(DV), ELEMS = 16 * (LK + LV);
    static constexpr uint32_t BYTES = ELEMS * 2;
    template <class T>
    __device__ static T *k(T *page, int row, int chunk) { return page + row * LK + page_chunk(KW, row, chunk) * 8; }
    template <class T>
    __device__ static T *v(T *page, int row, int chunk) { return page + 16 * LK + row * LV + page_chunk(DV, row, chunk) * 8; }
    // values of rows that nobody has written: a weight of zero does not hide what is not a number
    __device__ static void clear_values(__nv_bfloat16 *page, int from, int lane) {
        for (int e = from * (LV / 8) + lane; e < 16 * (LV / 8); e += 32) reinterpret_cast<uint4 *>(page + 16 * LK)[e] = make_uint4(0, 0, 0, 0);
    }
};

// Entries with several tokens (K / V are in the pages).  CTA = 64 rows of one key head (32 with two maps): four warps of 16 rows of
// one map, prepared on their way in; a fifth warp brings in tiles of KT keys, a bulk copy per page.  The second map's warps hand
// their rows over in shared memory.
template <int DK, int DV, int MAPS>
struct Tile {
    using P = Page<MAPS * DK, DV>;
    static constexpr int KT = 64, ST = 2, PAGES = KT / 16, LQ = DK + 8, ROWS = 64 / MAPS, BLOCKS = DV <= 128 ? 2 : 1;
    static constexpr size_t stage_elems = (size_t)PAGES * P::ELEMS, ring = ST * stage_elems * 2, hand = MAPS == 2 ? (size_t)ROWS * (DV + 8) * 4 : 0;
    static constexpr size_t smem = (ring > hand ? ring : hand) + (size_t)64 * LQ * 2;
};

// EXTRA: windows with kept tokens, sinks, norms over whole rows.
template <int DK, int DV, int MAPS, bool EXTRA>
__global__ void __launch_bounds__(160, (Tile<DK, DV, MAPS>::BLOCKS)) attn_tile_kernel(const AttnArgs a, const Seg *__restrict__ segs, const int2 *__restrict__ tiles, int qt, int pdl) {
    using T = Tile<DK, DV, MAPS>;
    using P = typename T::P;
    constexpr int LQ = T::LQ, KT = T::KT, ST = T::ST, PAGES = T::PAGES, NC = 128, LV = DV + 8, ROWS = T::ROWS;
    extern __shared__ __align__(128) uint8_t attn_smem[];
    __nv_bfloat16 *ring = reinterpret_cast<__nv_bfloat16 *>(attn_smem);  // stages of PAGES pages
    __nv_bfloat16 *qs = reinterpret_cast<__nv_bfloat16 *>(attn_smem + T::smem) - 64 * LQ;
    __shared__ __align__(8) uint64_t full[ST], empty[ST];
    __shared__ int s_abort_mem;
    volatile int *s_abort = &s_abort_mem;
    const int tid = threadIdx.x, lane = tid & 31, g = lane >> 2, wid = tid >> 5, map = wid / (ROWS / 16), warp = wid % (ROWS / 16);
    const int grp = a.heads / a.kv_heads, kvh = blockIdx.y, r0 = blockIdx.z * ROWS;
    if (pdl & 2) griddep_launch_dependents();
    const int2 tile = tiles[gridDim.x - 1 - blockIdx.x];  // the last tiles of a prompt see most keys
    const Seg sg = segs[tile.x];
    const int nt = min(qt, sg.T - tile.y), rows = nt * grp, row_base = sg.row0 + tile.y;
    if (r0 >= rows) return;
    const int p0 = sg.pos0 + tile.y, b0 = p0 + r0 / grp, p1 = p0 + (min(rows, r0 + ROWS) - 1) / grp;  // positions: of the tile, of the block's rows
    // keys in tiles: the kept ones when they lie apart, then those from the first one that the block's first row sees
    const int win = first_visible<EXTRA>(b0, a) / kBlockTokens * kBlockTokens, kept = EXTRA ? kept_apart(win, a) : 0, first = EXTRA && a.keep && !kept ? 0 : win;
    const int n_kept = (kept + KT - 1) / KT, n_tiles = n_kept + (p1 - first) / KT + 1;
    auto tile_key = [&](int it) { return it < n_kept ? it * KT : first + (it - n_kept) * KT; };
    if (tid == 0) {
        for (int s = 0; s < ST; s++) mbar_init(&full[s], 1), mbar_init(&empty[s], NC / 32);
        *s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    if (pdl & 1) griddep_wait();
    if (tid >= NC) {
        const __nv_bfloat16 *kv = reinterpret_cast<const __nv_bfloat16 *>(a.kv) + (size_t)kvh * P::ELEMS;
        auto lookup = [&](int it) {
            const int key = tile_key(it) + lane * 16;
            return lane < PAGES && it < n_tiles && key <= p1 ? page_of(a, sg.seq, key) : -1;
        };
        int phys = lookup(0), it = 0;
        for (; it < n_tiles; it++) {
            const int next = lookup(it + 1), s = it % ST;
            int ok = 1;
            const uint32_t pages = __popc(__ballot_sync(0xffffffffu, phys >= 0));
            if (lane == 0) {
                if (it >= ST) ok = mbar_wait_bounded(&empty[s], (it / ST - 1) & 1, a.status, s_abort);
                if (ok) mbar_expect_tx(&full[s], pages * P::BYTES);
            }
            if (!__shfl_sync(0xffffffffu, ok, 0)) break;
            if (phys >= 0) bulk_g2s(ring + s * T::stage_elems + lane * P::ELEMS, kv + (size_t)phys * a.kv_heads * P::ELEMS, P::BYTES, &full[s]);
            phys = next;
        }
        if (*s_abort && lane == 0)  // copies in flight still target this CTA's shared memory: a bounded chance to land
            for (int k = max(it - ST, 0); k < it; k++)
                for (uint32_t i = 0; i < (1u << 16) && !mbar_try_wait(&full[k % ST], (k / ST) & 1u); i++) {
                }
        return;
    }
    {
        constexpr int LANES = head_lanes(DK), PER = NC / LANES, N = 64 / PER;  // vectors at a time, rounds
        const __nv_bfloat16 *proj = reinterpret_cast<const __nv_bfloat16 *>(a.proj);
        const int piece = tid & (LANES - 1);
        auto source = [&](int v, int &row, int &h) {  // vector v = row of the block, map
            const int r = r0 + v / MAPS, t = r / grp;
            h = kvh * grp + r % grp, row = row_base + t;
            return r < rows ? proj + (size_t)row * a.ldp + a.q_off + (h * MAPS + v % MAPS) * DK : nullptr;
        };
        uint4 raw[N];
#pragma unroll
        for (int n = 0; n < N; n++) {
            int row, h;
            const __nv_bfloat16 *src = source(n * PER + tid / LANES, row, h);
            raw[n] = src && piece * 8 < DK ? *reinterpret_cast<const uint4 *>(src + piece * 8) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int n = 0; n < N; n++) {
            const int v = n * PER + tid / LANES;
            if (a.prepared()) {
                int row, h;
                const __nv_bfloat16 *src = source(v, row, h);
                if (!src) row = row_base, h = 0;
                float x[8];
                load8(reinterpret_cast<const __nv_bfloat16 *>(&raw[n]), x);
                prepare_head(x, src ? src : proj, piece, LANES, head_prep<EXTRA>(a, false, row, h, EXTRA && a.whole_rows ? a.row_inv[row].x : 1.f));
                store8(reinterpret_cast<__nv_bfloat16 *>(&raw[n]), x);
            }
            if (piece * 8 < DK) *reinterpret_cast<uint4 *>(qs + (v % MAPS * ROWS + v / MAPS) * LQ + piece * 8) = raw[n];
        }
        named_bar_sync(1, NC);
    }
    int lo[2], hi[2], rt[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int r = r0 + warp * 16 + g + 8 * e;
        rt[e] = r < rows ? r : -1;
        hi[e] = p0 + (r < rows ? r : r0) / grp;
        lo[e] = first_visible<EXTRA>(hi[e], a);
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    auto qfrag = [&](int kk, uint32_t (&f)[4]) {
        ldmatrix_x4(f, qs + (size_t)(map * ROWS + warp * 16 + (lane & 15)) * LQ + kk * 16 + (lane >> 4) * 8);
    };
    const float sl = a.scale * 1.4426950408889634f;
    const int vis_lo = first_visible<EXTRA>(p1, a);
    for (int it = 0; it < n_tiles; it++) {
        const int s = it % ST, kb = tile_key(it);
        const bool apart = EXTRA && it < n_kept;
        if (!__all_sync(0xffffffffu, mbar_wait_bounded(&full[s], (it / ST) & 1, a.status, s_abort))) break;
        __nv_bfloat16 *stage = ring + s * T::stage_elems;
        if (kb + KT > p1 + 1) {  // every warp clears what it is going to read
#pragma unroll
            for (int i = 0; i < PAGES; i++)
                if (kb + 16 * i + 15 > p1) P::clear_values(stage + i * P::ELEMS, max(p1 + 1 - kb - 16 * i, 0), lane);
            __syncwarp();
        }
        auto kat = [&](int r, int c) { return P::k(stage + (r >> 4) * P::ELEMS, r & 15, map * (DK / 8) + c); };
        auto vat = [&](int r, int c) { return P::v(stage + (r >> 4) * P::ELEMS, r & 15, c); };
        if (EXTRA) {
            const int from[2] = {apart ? 0 : lo[0], apart ? 0 : lo[1]}, to[2] = {apart ? kept - 1 : hi[0], apart ? kept - 1 : hi[1]};
            attend_tile<DK, DV, KT, true>(qfrag, kat, vat, kb, apart || kb + KT - 1 > b0 || kb < vis_lo, from, to, a.keep, sl, m, l, o, lane);
        } else {
            attend_tile<DK, DV, KT, false>(qfrag, kat, vat, kb, kb + KT - 1 > b0 || kb < vis_lo, lo, hi, 0, sl, m, l, o, lane);
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(&empty[s]);
    }
    float f[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        f[e] = l[e] > 0.f ? 1.f / l[e] : 0.f;
        if (EXTRA && a.sink && rt[e] >= 0) {  // its share: relative to the larger of the two scores
            const float sk = a.sink[kvh * grp + rt[e] % grp] * 1.4426950408889634f, mn = fmaxf(m[e], sk), w = fast_exp2(m[e] - mn);
            f[e] = w / (l[e] * w + fast_exp2(sk - mn));
        }
    }
    if (MAPS == 2) {
        float *other = reinterpret_cast<float *>(ring);  // [ROWS][DV + 8]
        named_bar_sync(1, NC);  // every warp is done with the stages
        const int t2 = 2 * (lane & 3);
        if (map == 1) {
#pragma unroll
            for (int e = 0; e < 2; e++)
#pragma unroll
                for (int n = 0; n < DV / 8; n++)
                    *reinterpret_cast<float2 *>(other + (warp * 16 + g + 8 * e) * LV + n * 8 + t2) = make_float2(o[n][2 * e] * f[e], o[n][2 * e + 1] * f[e]);
        }
        named_bar_sync(1, NC);
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
// fourth page of its CTA through its own ring of bulk copies (no block barrier in the loop), and the partial softmax states meet
// through cluster shared memory.  The query rows are the heads of the group times the maps: with two maps a row is zero outside its
// own map's half of the key, so one product scores both.  With one map CTA r of the cluster finishes its share of the head's
// columns, with two a warp somewhere in the cluster finishes a head.  With FUSED the token's own K and V are not in the pages yet:
// the CTA that owns the last page prepares and writes them, and patches its copy of the page; earlier pages are requested before
// the wait for the launch in front.
template <int DK, int DV>
struct Single {
    using P = Page<DK, DV>;
    static constexpr int ST = 4 * 6 * P::BYTES <= 104 * 1024 ? 6 : (4 * 4 * P::BYTES <= 104 * 1024 ? 4 : (4 * 3 * P::BYTES <= 104 * 1024 ? 3 : 2));
    static constexpr int PW = DV + 4, LQ = DK + 8;
    static constexpr size_t ring_bytes = 4 * ST * (size_t)P::BYTES, part_bytes = sizeof(float) * 4 * 16 * PW, front = ring_bytes > part_bytes ? ring_bytes : part_bytes;
    static constexpr size_t merged_bytes = sizeof(float) * 16 * PW, query_bytes = (size_t)2 * (16 * LQ + DK + DV);
    static constexpr size_t smem = front + (merged_bytes > query_bytes ? merged_bytes : query_bytes);
};

template <int DK, int DV>  // DK: of all maps together
__global__ void __launch_bounds__(128) attn_single_kernel(const AttnArgs a, const Seg *__restrict__ segs, const int *__restrict__ singles, int row_blocks,
                                                          int fused, int pdl) {
    using S = Single<DK, DV>;
    using P = typename S::P;
    constexpr int LQ = S::LQ, ST = S::ST, PW = S::PW, CV = DV / 8;
    extern __shared__ __align__(128) uint8_t attn_smem[];
    __nv_bfloat16 *ring = reinterpret_cast<__nv_bfloat16 *>(attn_smem);        // [4 warps][ST] pages
    float *part = reinterpret_cast<float *>(attn_smem);                        // [4 warps][16][m, l, -, -, o[DV]], after the loop
    float *merged = reinterpret_cast<float *>(attn_smem + S::front);           // [16][m, l, -, -, o[DV]] of this CTA, after the loop
    __nv_bfloat16 *qs = reinterpret_cast<__nv_bfloat16 *>(attn_smem + S::front), *own = qs + 16 * LQ;  // query rows [16][LQ]; the token's [K | V]
    __shared__ __align__(8) uint64_t full[4][ST];
    __shared__ float2 red[4];
    __shared__ int s_abort_mem;
    volatile int *s_abort = &s_abort_mem;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = 2 * (lane & 3);
    const int nsplit = gridDim.x, split = blockIdx.x, maps = a.maps, hpb = 16 / maps, dk = DK / maps;
    const int rb = blockIdx.y % row_blocks, kvh = blockIdx.y / row_blocks, grp = a.heads / a.kv_heads, h0 = kvh * grp + rb * hpb, nh = min(hpb, grp - rb * hpb);
    if (pdl & 2) griddep_launch_dependents();
    const Seg sg = segs[singles[blockIdx.z]];
    // pages in order: the kept ones when they lie apart, then those from the first one seen; this CTA has [pg0, pg1) of them
    const int p = sg.pos0, row = sg.row0, first = first_visible(p, a), win_page = first / kBlockTokens, kept = kept_apart(win_page * kBlockTokens, a);
    const int lo_page = a.keep && !kept ? 0 : win_page, n_kept = (kept + kBlockTokens - 1) / kBlockTokens, last = p / kBlockTokens, n_pages = n_kept + last - lo_page + 1;
    const int pg0 = split * n_pages / nsplit, pg1 = (split + 1) * n_pages / nsplit;
    auto page_at = [&](int i) { return i < n_kept ? i : i - n_kept + lo_page; };
    __nv_bfloat16 *kv = reinterpret_cast<__nv_bfloat16 *>(a.kv) + (size_t)kvh * P::ELEMS;
    if (lane == 0) {
        for (int s = 0; s < ST; s++) mbar_init(&full[warp][s], 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (tid == 0) *s_abort = 0;
    for (int e = tid; e < 16 * LQ / 8; e += 128) reinterpret_cast<uint4 *>(qs)[e] = make_uint4(0, 0, 0, 0);
    __syncthreads();
    __nv_bfloat16 *mine = ring + (size_t)warp * ST * P::ELEMS;
    // physical blocks of this warp's next 32 pages, a page per lane: one trip to the table instead of one per page
    int blocks = -1;
    auto load = [&](int i) {  // the i-th page of this warp
        const int pg = pg0 + warp + 4 * i;
        if ((i & 31) == 0) {
            const int at = pg + 4 * lane;
            blocks = at < pg1 ? page_of(a, sg.seq, page_at(at) * kBlockTokens) : -1;
        }
        const int phys = __shfl_sync(0xffffffffu, blocks, i & 31);
        if (pg < pg1 && lane == 0) {
            mbar_expect_tx(&full[warp][i % ST], phys >= 0 ? P::BYTES : 0);
            if (phys >= 0) bulk_g2s(mine + (size_t)(i % ST) * P::ELEMS, kv + (size_t)phys * a.kv_heads * P::ELEMS, P::BYTES, &full[warp][i % ST]);
        }
    };
    const bool append = fused && split == nsplit - 1;
    if (fused) {
#pragma unroll
        for (int i = 0; i < ST; i++) load(i);
    }
    if (pdl & 1) griddep_wait();
    if (!fused) {
#pragma unroll
        for (int i = 0; i < ST; i++) load(i);
    }
    const __nv_bfloat16 *proj = reinterpret_cast<const __nv_bfloat16 *>(a.proj) + (size_t)row * a.ldp;
    {
        float2 inv = make_float2(1.f, 1.f);
        if (a.whole_rows) {
            if (fused) {
                inv = row_rms(proj, a, red);
            } else {
                inv = a.row_inv[row];
            }
        }
        // heads of the group, then (with the last page) the key's maps
        const int lanes = head_lanes(dk), piece = tid & (lanes - 1), slots = 128 / lanes, nq = nh * maps;
        const int phys = append ? page_of(a, sg.seq, p) : -1, total = nq + (append ? maps : 0), r = p % kBlockTokens;
        __nv_bfloat16 *page = kv + (size_t)max(phys, 0) * a.kv_heads * P::ELEMS;
        for (int v0 = 0; v0 < total; v0 += slots) {
            const int v = v0 + tid / lanes;
            const bool load = v < total && piece * 8 < dk, key = v >= nq;
            const __nv_bfloat16 *src = proj + (key ? a.k_off + (kvh * maps + min(v - nq, maps - 1)) * dk : a.q_off + (h0 * maps + v) * dk);
            float x[8];
            if (load) load8(src + piece * 8, x);
            else {
#pragma unroll
                for (int e = 0; e < 8; e++) x[e] = 0.f;
            }
            if (a.prepared()) prepare_head(x, src, piece, lanes, head_prep<true>(a, key, row, key ? kvh : min(h0 + v, a.heads - 1), key ? inv.y : inv.x));
            if (!load) continue;
            if (key) {
                const int c = (v - nq) * (dk / 8) + piece;
                store8(own + c * 8, x);
                if (phys >= 0) store8(P::k(page, r, c), x);
            } else {
                store8(qs + ((v % maps) * hpb + v / maps) * LQ + (v % maps) * dk + piece * 8, x);
            }
        }
        if (append)
            for (int c = tid; c < CV; c += 128) {
                if (values_line_up(a, c * 8)) {
                    float x[8];
                    load_values<__nv_bfloat16>(a, row, kvh, c * 8, x);
                    store8(own + DK + c * 8, x);
                } else {
#pragma unroll 1
                    for (int e = 0; e < 8; e++) act_store(own + DK + c * 8 + e, load_value<__nv_bfloat16>(a, row, kvh, c * 8 + e));
                }
                if (phys >= 0) *reinterpret_cast<uint4 *>(P::v(page, r, c)) = *reinterpret_cast<const uint4 *>(own + DK + c * 8);
            }
        __syncthreads();
    }
    uint32_t q[DK / 16][4];
#pragma unroll
    for (int kk = 0; kk < DK / 16; kk++) ldmatrix_x4(q[kk], qs + (size_t)(lane & 15) * LQ + kk * 16 + (lane >> 4) * 8);
    auto qfrag = [&](int kk, uint32_t (&f)[4]) { f[0] = q[kk][0], f[1] = q[kk][1], f[2] = q[kk][2], f[3] = q[kk][3]; };
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    const float sl = a.scale * 1.4426950408889634f;
    for (int i = 0; pg0 + warp + 4 * i < pg1; i++) {
        const bool apart = pg0 + warp + 4 * i < n_kept;
        const int pg = page_at(pg0 + warp + 4 * i), kb = pg * kBlockTokens;
        if (!__all_sync(0xffffffffu, mbar_wait_bounded(&full[warp][i % ST], (i / ST) & 1, a.status, s_abort))) break;
        __nv_bfloat16 *page = mine + (size_t)(i % ST) * P::ELEMS;
        if (pg == last) {
            const int r = p % kBlockTokens;
            P::clear_values(page, r + (fused ? 0 : 1), lane);
            __syncwarp();
            if (fused) {
                for (int c = lane; c < DK / 8; c += 32) *reinterpret_cast<uint4 *>(P::k(page, r, c)) = *reinterpret_cast<const uint4 *>(own + c * 8);
                for (int c = lane; c < CV; c += 32) *reinterpret_cast<uint4 *>(P::v(page, r, c)) = *reinterpret_cast<const uint4 *>(own + DK + c * 8);
                __syncwarp();
            }
        }
        auto kat = [&](int r, int c) { return P::k(page, r, c); };
        auto vat = [&](int r, int c) { return P::v(page, r, c); };
        const int from = apart ? 0 : first, to = apart ? kept - 1 : p, lo[2] = {from, from}, hi[2] = {to, to};
        attend_tile<DK, DV, 16, true>(qfrag, kat, vat, kb, kb < from || kb + 15 > to, lo, hi, a.keep, sl, m, l, o, lane);
        __syncwarp();
        load(i + ST);
    }
    if (*s_abort && lane == 0)  // copies in flight still target this CTA's shared memory: a bounded chance to land
        for (int i = 0; pg0 + warp + 4 * i < pg1; i++)
            for (uint32_t k = 0; k < (1u << 14) && !mbar_try_wait(&full[warp][i % ST], (i / ST) & 1u); k++) {
            }
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
            const float sk = a.sink ? a.sink[h0 + r] * 1.4426950408889634f : -INFINITY;
            float mx = sk, sum = 0.f, acc = 0.f;
            if (nsplit == 1) {
                const float ms = merged[r * PW];
                mx = fmaxf(mx, ms);
                const float f = a.sink && ms != -INFINITY ? fast_exp2(ms - mx) : 1.f;
                sum = f * merged[r * PW + 1], acc = f * merged[r * PW + 4 + c];
            } else {
                for (int s = 0; s < nsplit; s++) mx = fmaxf(mx, ld_cluster_f32(merged + r * PW, (uint32_t)s));
                for (int s = 0; s < nsplit; s++) {
                    const float ms = ld_cluster_f32(merged + r * PW, (uint32_t)s), f = ms == -INFINITY ? 0.f : fast_exp2(ms - mx);
                    sum += f * ld_cluster_f32(merged + r * PW + 1, (uint32_t)s), acc += f * ld_cluster_f32(merged + r * PW + 4 + c, (uint32_t)s);
                }
            }
            if (a.sink) sum += fast_exp2(sk - mx);
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
constexpr HeadSizes kHeadSizes[] = {{1, 32, 32},  {1, 64, 32},  {1, 64, 64},  {1, 96, 64},  {1, 96, 96},  {1, 128, 64}, {1, 128, 128}, {1, 192, 192}, {1, 256, 256},
                                    {2, 32, 32},  {2, 32, 64},  {2, 64, 64},  {2, 64, 96},  {2, 64, 128}, {2, 96, 192},  {2, 128, 128}, {2, 128, 256}};

bool attn_padded_head(int dim, int vdim, int maps, int *DK, int *DV) {
    int best = 0;
    for (const HeadSizes &s : kHeadSizes)
        if (s.maps == maps && dim > 0 && vdim > 0 && dim <= s.DK && vdim <= s.DV && (!best || s.DK + s.DV < best)) best = s.DK + s.DV, *DK = s.DK, *DV = s.DV;
    return best > 0;
}
int attn_query_tile(int heads, int kv_heads) { return std::max(1, 64 / (heads / kv_heads)); }

// Threads of a row's preparation: one block, or several of 256.
static void prep_shape(const AttnArgs &a, bool queries, int rows, dim3 *grid, dim3 *block) {
    const int threads = ((queries ? a.heads * a.maps : 0) + a.kv_heads * (a.maps + 1)) * head_lanes(a.DK);
    *block = dim3((unsigned)std::min(256, (threads + 31) / 32 * 32)), *grid = dim3((unsigned)rows, a.wide() ? 1u : (threads + block->x - 1) / block->x);
}

template <class AT>
static int32_t rows_attention(const StepDesc &d, const AttnArgs &a, cudaStream_t st) {
    dim3 grid, block;
    prep_shape(a, a.prepared(), d.rows, &grid, &block);
    if (a.wide()) attn_prep_kernel<AT, true><<<grid, block, 0, st>>>(a, d.seq, d.pos, a.prepared(), 0);
    else attn_prep_kernel<AT, false><<<grid, block, 0, st>>>(a, d.seq, d.pos, a.prepared(), 0);
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
        using T = Tile<DK, DV, MAPS>;
        prep_shape(a, false, d.rows, &cfg.gridDim, &cfg.blockDim);
        cfg.dynamicSmemBytes = 0, cfg.numAttrs = (unsigned)early(0);
        JGPT_CUDA_TRY(a.wide() ? cudaLaunchKernelEx(&cfg, attn_prep_kernel<__nv_bfloat16, true>, a, d.seq, d.pos, 0, pdl)
                               : cudaLaunchKernelEx(&cfg, attn_prep_kernel<__nv_bfloat16, false>, a, d.seq, d.pos, 0, pdl));
        auto tiles = [&](auto kern, int &set_for) -> int32_t {
            if (int32_t rc = opt_in(kern, T::smem, set_for)) return rc;
            cfg.gridDim = dim3((unsigned)d.n_tiles, (unsigned)a.kv_heads, (unsigned)((d.qt * grp + T::ROWS - 1) / T::ROWS)), cfg.blockDim = dim3(160);
            cfg.dynamicSmemBytes = T::smem, cfg.numAttrs = (unsigned)early(0);
            JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, kern, a, d.segs, d.tiles, d.qt, pdl));
            return JGPT_OK;
        };
        static thread_local int plain_for = -1, extra_for = -1;
        if constexpr (MAPS == 1) {
            if (a.extra()) {
                if (int32_t rc = tiles(attn_tile_kernel<DK, DV, MAPS, true>, extra_for)) return rc;
            } else if (int32_t rc = tiles(attn_tile_kernel<DK, DV, MAPS, false>, plain_for)) {
                return rc;
            }
        } else if (int32_t rc = tiles(attn_tile_kernel<DK, DV, MAPS, false>, plain_for)) {
            return rc;
        }
    }
    if (d.n_singles) {
        static thread_local int set_for = -1;
        if (int32_t rc = opt_in(attn_single_kernel<KW, DV>, (Single<KW, DV>::smem), set_for)) return rc;
        const int row_blocks = (grp * MAPS + 15) / 16, ctas = d.n_singles * a.kv_heads * row_blocks;
        const int range = a.window > 0 ? a.window + a.keep : a.chunk, keys = range > 0 ? std::min(range, d.max_len) : d.max_len, pages = keys / kBlockTokens + 1;
        int split = 1;  // every warp keeps two pages, the grid stays around two CTAs per SM
        while (split < 8 && ctas * split * 2 <= 2 * a.sm_count && pages >= split * 2 * 8) split *= 2;
        int na = early(0);
        if (split > 1) {
            attr[na].id = cudaLaunchAttributeClusterDimension;
            attr[na].val.clusterDim.x = (unsigned)split, attr[na].val.clusterDim.y = 1, attr[na].val.clusterDim.z = 1;
            na++;
        }
        cfg.gridDim = dim3((unsigned)split, (unsigned)(a.kv_heads * row_blocks), (unsigned)d.n_singles), cfg.blockDim = dim3(128);
        cfg.dynamicSmemBytes = (Single<KW, DV>::smem), cfg.numAttrs = (unsigned)na;
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
