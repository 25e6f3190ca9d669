// Routing of the mixture of experts: a token's experts and their weights from its router logits, the rows of every expert, and the
// row tiles of the experts' products.
//
// One launch: a warp per token picks its experts, a block counts its tokens' picks and takes places in the experts' lists (lists
// have room for every row, since a token picks an expert once); the block that finishes last turns the counts into offsets and
// tiles and leaves the counters at zero.  Places depend on the order of
// arrival, results do not: every row of a product stands alone.
#include "mixers.cuh"
#include "ptx.cuh"

namespace jgpt {
namespace mix {

constexpr unsigned kAll = 0xffffffffu;
constexpr int kRouteWarps = 8;

__device__ __forceinline__ int warp_scan(int v) {  // inclusive
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
        const int o = __shfl_up_sync(kAll, v, off);
        if (lane >= off) v += o;
    }
    return v;
}
// Orders like the float, never 0: 0 stands for out of the question.
__device__ __forceinline__ uint32_t order_key(float v) {
    const uint32_t u = __float_as_uint(v);
    return u & 0x80000000u ? max(~u, 1u) : u | 0x80000000u;
}

// The warp's best key and its index, the lowest one among equals; -1: no key but zeros.
__device__ __forceinline__ int best_of_warp(uint32_t key, int at) {
    const uint32_t top = __reduce_max_sync(kAll, key);
    return top ? (int)__reduce_min_sync(kAll, key == top ? (unsigned)at : kAll) : -1;
}

// Experts of one token by one warp, which holds outputs lane + 32 i: lane s gets the s-th choice (-1: none) and its weight.
// group: a word of shared memory per group.
template <int NPL>
__device__ __forceinline__ void choose_experts(const RouteArgs &a, const float *logits, uint32_t *group, int &expert, float &weight) {
    const int lane = threadIdx.x & 31, E = a.experts + a.identity, size = E / a.groups;
    float score[NPL], mx = -INFINITY, sum = 0.f;
    uint32_t key[NPL];
#pragma unroll
    for (int i = 0; i < NPL; i++) score[i] = lane + 32 * i < E ? logits[lane + 32 * i] : -INFINITY, mx = fmaxf(mx, score[i]);
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(kAll, mx, off));
#pragma unroll
    for (int i = 0; i < NPL; i++) score[i] = expf(score[i] - mx), sum += score[i];
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) sum += __shfl_xor_sync(kAll, sum, off);
    const float inv = 1.f / sum;
#pragma unroll
    for (int i = 0; i < NPL; i++) score[i] *= inv, key[i] = lane + 32 * i < E ? order_key(score[i] + __ldg(a.correction + lane + 32 * i)) : 0;
    if (a.keep < a.groups) {
        for (int g = lane; g < a.groups; g += 32) group[g] = 0;
        __syncwarp();
        int mine[NPL];
#pragma unroll
        for (int i = 0; i < NPL; i++) {
            mine[i] = lane + 32 * i < E ? (lane + 32 * i) / size : 0;
            if (key[i]) atomicMax(group + mine[i], key[i]);
        }
        __syncwarp();
        for (int k = 0; k < a.keep; k++) {
            uint32_t top = 0;
            int at = 0;
            for (int g = lane; g < a.groups; g += 32)
                if (group[g] > top) top = group[g], at = g;
            const int taken = best_of_warp(top, at);
            if (taken >= 0 && (taken & 31) == lane) group[taken] = 0;
        }
        __syncwarp();
#pragma unroll
        for (int i = 0; i < NPL; i++)
            if (group[mine[i]]) key[i] = 0;  // a group that was not taken
        __syncwarp();                        // the words are free for the next token
    }
    expert = -1, weight = 0.f;
    float total = 0.f;
    for (int s = 0; s < a.top; s++) {
        uint32_t top = 0;
        int at = 0;
        float w = 0.f;
#pragma unroll
        for (int i = 0; i < NPL; i++)
            if (key[i] > top) top = key[i], at = lane + 32 * i, w = score[i];
        const int taken = best_of_warp(top, at);
        if (taken < 0) break;
        w = __shfl_sync(kAll, w, taken & 31), total += w;
        if (lane == s) expert = taken, weight = w;
#pragma unroll
        for (int i = 0; i < NPL; i++)
            if (lane + 32 * i == taken) key[i] = 0;
    }
    weight /= total + 1e-20f;
}

// Offsets and tiles from the experts' counts, by one warp.
template <class Count>
__device__ __forceinline__ void plan_tiles(const RouteArgs &a, const Count &count) {
    const int lane = threadIdx.x & 31;
    int rows = 0, tiles = 0;
    for (int e0 = 0; e0 < a.experts; e0 += 32) {
        const int e = e0 + lane;
        const int n = e < a.experts ? min(count(e), a.cap) : 0, nt = (n + a.tile_rows - 1) / a.tile_rows;
        const int rs = warp_scan(n), ts = warp_scan(nt), row0 = rows + rs - n, t0 = tiles + ts - nt;
        if (e < a.experts) {
            a.offsets[e] = row0;
            for (int t = 0; t < nt; t++)
                if (t0 + t < a.max_tiles)
                    a.tiles[t0 + t] = nt::RowTile{e, row0 + t * a.tile_rows, min(row0 + n, row0 + (t + 1) * a.tile_rows), e * a.cap + t * a.tile_rows};
        }
        rows += __shfl_sync(kAll, rs, 31), tiles += __shfl_sync(kAll, ts, 31);
    }
    if (lane == 0) *a.n_tiles = min(tiles, a.max_tiles);
}

template <int NPL>
__global__ void __launch_bounds__(32 * kRouteWarps) route_kernel(const RouteArgs a, int rows, int per_block, int pdl) {
    extern __shared__ uint32_t route_smem[];
    __shared__ int last;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, E = a.experts + a.identity;
    const int r0 = blockIdx.x * per_block, n = min(per_block, rows - r0);
    uint32_t *group = route_smem + warp * a.groups;
    int *counts = reinterpret_cast<int *>(route_smem) + kRouteWarps * a.groups, *base = counts + a.experts;
    RouteSlot *slots = reinterpret_cast<RouteSlot *>(base + a.experts);
    if (pdl & 2) griddep_launch_dependents();
    for (int e = tid; e < a.experts; e += blockDim.x) counts[e] = 0;
    if (pdl & 1) griddep_wait();
    __syncthreads();
    for (int t = warp; t < n; t += kRouteWarps) {
        const float *logits = a.logits + (size_t)(r0 + t) * a.ld;
        int expert;
        float weight;
        choose_experts<NPL>(a, logits, group, expert, weight);
        const bool real = expert >= 0 && expert < a.experts;
        if (lane < a.top) slots[t * a.top + lane] = RouteSlot{real ? expert : -1, real ? atomicAdd(counts + expert, 1) : -1, real ? weight : 0.f};
        float id = expert >= a.experts ? weight : 0.f;
#pragma unroll
        for (int off = 16; off >= 1; off >>= 1) id += __shfl_xor_sync(kAll, id, off);
        if (lane == 0) a.row_weights[r0 + t] = make_float2(id, a.shared ? 1.f / (1.f + expf(-logits[E])) : 0.f);
    }
    __syncthreads();
    const bool alone = gridDim.x == 1;
    for (int e = tid; e < a.experts; e += blockDim.x) base[e] = alone || counts[e] == 0 ? 0 : atomicAdd(a.counts + e, counts[e]);
    __syncthreads();
    for (int i = tid; i < n * a.top; i += blockDim.x) {
        RouteSlot s = slots[i];
        if (s.expert >= 0) {
            s.rank += base[s.expert];
            if (s.rank < a.cap) a.list[(size_t)s.expert * a.cap + s.rank] = r0 + i / a.top;
        }
        a.slots[(size_t)r0 * a.top + i] = s;
    }
    if (alone) {
        if (warp == 0) plan_tiles(a, [&](int e) { return counts[e]; });
        return;
    }
    if (tid == 0) __threadfence(), last = atomicAdd(a.ticket, 1) == (int)gridDim.x - 1;
    __syncthreads();
    if (!last || warp != 0) return;
    __threadfence();
    if (lane == 0) *a.ticket = 0;
    plan_tiles(a, [&](int e) { return atomicExch(a.counts + e, 0); });
}

// A block per 16 rows of a tile.  (Nothing here is __restrict__: reads of what counts as constant may move up past the wait.)
__global__ void __launch_bounds__(256) moe_gather_kernel(const RouteArgs a, const uint4 *h, uint4 *out, int chunks, int pdl) {
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    if ((int)blockIdx.x >= *a.n_tiles) return;
    const nt::RowTile t = a.tiles[blockIdx.x];
    const int row0 = t.row0 + blockIdx.y * 16, n = min(16, t.row_end - row0), *from = a.list + t.src0 + blockIdx.y * 16;
    for (int i0 = threadIdx.x; i0 < n * chunks; i0 += 8 * 256) {
        uint4 x[8];
#pragma unroll
        for (int k = 0; k < 8; k++)
            if (const int i = i0 + 256 * k; i < n * chunks) x[k] = h[(size_t)from[i / chunks] * chunks + i % chunks];
#pragma unroll
        for (int k = 0; k < 8; k++)
            if (const int i = i0 + 256 * k; i < n * chunks) out[(size_t)row0 * chunks + i] = x[k];
    }
}

template <class... Args>
static int32_t launch(void (*kern)(Args...), dim3 grid, int threads, size_t smem, int pdl, cudaStream_t st, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = grid, cfg.blockDim = dim3((unsigned)threads), cfg.dynamicSmemBytes = smem, cfg.stream = st;
    cfg.attrs = attr, cfg.numAttrs = (pdl & 1) ? 1 : 0;
    JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, kern, args...));
    return JGPT_OK;
}

int32_t launch_route(const RouteArgs &a, int rows, int pdl, cudaStream_t st) {
    // few tokens: one per warp, and one block for as many as it has warps; many: four per warp
    const int per_block = rows <= 512 ? kRouteWarps : 4 * kRouteWarps, E = a.experts + a.identity;
    const size_t smem = 4 * ((size_t)kRouteWarps * a.groups + 2 * (size_t)a.experts) + sizeof(RouteSlot) * (size_t)per_block * a.top;
    JGPT_REQUIRE(smem <= 47 * 1024 && a.top <= 32 && E <= 1024, JGPT_ERR_UNSUPPORTED, "%d router outputs, %d chosen", E, a.top);
    auto run = [&](auto kern) { return launch(kern, dim3((unsigned)((rows + per_block - 1) / per_block)), 32 * kRouteWarps, smem, pdl, st, a, rows, per_block, pdl); };
    if (E <= 32) return run(route_kernel<1>);
    if (E <= 64) return run(route_kernel<2>);
    if (E <= 128) return run(route_kernel<4>);
    return E <= 256 ? run(route_kernel<8>) : run(route_kernel<32>);
}

int32_t launch_moe_gather(const RouteArgs &a, const void *h, void *out, int ld, int pdl, cudaStream_t st) {
    return launch(moe_gather_kernel, dim3((unsigned)a.max_tiles, (unsigned)((a.tile_rows + 15) / 16)), 256, 0, pdl, st, a,
                  reinterpret_cast<const uint4 *>(h), reinterpret_cast<uint4 *>(out), ld / 8, pdl);
}

}  // namespace mix
}  // namespace jgpt
