// Routing of the mixture of experts: a token's experts and their weights from its router logits, the rows of every expert, and the
// row tiles of the experts' products.
//
// One launch: a warp per token picks its experts and takes a place in each one's list (lists have room for every row, since a token
// picks an expert once); the block that finishes last turns the counts into offsets and tiles and leaves the counters at zero.
// Places depend on the order of arrival, results do not: every row of a product stands alone.
#include "mixers.cuh"
#include "ptx.cuh"

namespace jgpt {
namespace mix {

constexpr int kRouteWarps = 4;

// The largest value of the warp's v and its index, the lowest one among equals.
__device__ __forceinline__ void warp_best(float &v, int &i) {
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, off);
        const int oi = __shfl_xor_sync(0xffffffffu, i, off);
        if (ov > v || (ov == v && oi < i)) v = ov, i = oi;
    }
}
__device__ __forceinline__ int warp_scan(int v) {  // inclusive
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
        const int o = __shfl_up_sync(0xffffffffu, v, off);
        if (lane >= off) v += o;
    }
    return v;
}

// Experts of one token by one warp: lane s gets the s-th choice and its weight.  score, choice: E values of shared memory each.
__device__ __forceinline__ void choose_experts(const RouteArgs &a, const float *logits, float *score, float *choice, float *group, int &expert, float &weight) {
    const int lane = threadIdx.x & 31, E = a.experts + a.identity, size = E / a.groups;
    float mx = -INFINITY, sum = 0.f;
    for (int e = lane; e < E; e += 32) score[e] = logits[e], mx = fmaxf(mx, score[e]);
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    for (int e = lane; e < E; e += 32) score[e] = expf(score[e] - mx), sum += score[e];
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
    for (int e = lane; e < E; e += 32) score[e] /= sum, choice[e] = score[e] + a.correction[e];
    __syncwarp();
    if (a.keep < a.groups) {
        for (int g = lane; g < a.groups; g += 32) {
            float best = -INFINITY;
            for (int e = g * size; e < (g + 1) * size; e++) best = fmaxf(best, choice[e]);
            group[g] = best;
        }
        __syncwarp();
        for (int k = 0; k < a.keep; k++) {
            float v = -INFINITY;
            int at = a.groups;
            for (int g = lane; g < a.groups; g += 32)
                if (group[g] > v) v = group[g], at = g;
            warp_best(v, at);
            if (lane == 0 && at < a.groups) group[at] = __int_as_float(0x7fc00000);  // NaN: taken, and no larger than anything
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
            if (!isnan(group[e / size])) choice[e] = -INFINITY;
        __syncwarp();
    }
    expert = -1, weight = 0.f;
    float total = 0.f;
    for (int s = 0; s < a.top; s++) {
        float v = -INFINITY;
        int at = E;
        for (int e = lane; e < E; e += 32)
            if (choice[e] > v) v = choice[e], at = e;
        warp_best(v, at);
        if (at >= E) break;  // nothing comparable left
        const float w = score[at];
        total += w;
        if (lane == s) expert = at, weight = w;
        if (lane == 0) choice[at] = -INFINITY;
        __syncwarp();
    }
    weight /= total + 1e-20f;
}

// Offsets and tiles from the counts, by one block; the counters go back to zero.
__device__ __forceinline__ void plan_tiles(const RouteArgs &a) {
    const int lane = threadIdx.x & 31;
    if (threadIdx.x >= 32) return;
    int rows = 0, tiles = 0;
    for (int e0 = 0; e0 < a.experts; e0 += 32) {
        const int e = e0 + lane;
        const int n = e < a.experts ? min(atomicExch(a.counts + e, 0), a.cap) : 0, nt = (n + a.tile_rows - 1) / a.tile_rows;
        const int rs = warp_scan(n), ts = warp_scan(nt), row0 = rows + rs - n, t0 = tiles + ts - nt;
        if (e < a.experts) {
            a.offsets[e] = row0;
            for (int t = 0; t < nt; t++)
                if (t0 + t < a.max_tiles)
                    a.tiles[t0 + t] = nt::RowTile{e, row0 + t * a.tile_rows, min(row0 + n, row0 + (t + 1) * a.tile_rows), e * a.cap + t * a.tile_rows};
        }
        rows += __shfl_sync(0xffffffffu, rs, 31), tiles += __shfl_sync(0xffffffffu, ts, 31);
    }
    if (lane == 0) *a.n_tiles = min(tiles, a.max_tiles);
}

__global__ void __launch_bounds__(32 * kRouteWarps) route_kernel(const RouteArgs a, int rows, int pdl) {
    extern __shared__ float route_smem[];
    __shared__ int last;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, E = a.experts + a.identity, r = blockIdx.x * kRouteWarps + warp;
    float *score = route_smem + warp * (2 * E + a.groups), *choice = score + E, *group = choice + E;
    if (pdl & 2) griddep_launch_dependents();
    if (pdl & 1) griddep_wait();
    if (r < rows) {
        int expert;
        float weight;
        const float *logits = a.logits + (size_t)r * a.ld;
        choose_experts(a, logits, score, choice, group, expert, weight);
        const bool real = lane < a.top && expert >= 0 && expert < a.experts;
        int rank = -1;
        if (real) {
            rank = atomicAdd(a.counts + expert, 1);
            if (rank < a.cap) a.list[(size_t)expert * a.cap + rank] = r;
        }
        float id = lane < a.top && expert >= a.experts ? weight : 0.f;
#pragma unroll
        for (int off = 16; off >= 1; off >>= 1) id += __shfl_xor_sync(0xffffffffu, id, off);
        if (lane < a.top) a.slots[(size_t)r * a.top + lane] = RouteSlot{real ? expert : -1, rank, real ? weight : 0.f};
        if (lane == 0) a.row_weights[r] = make_float2(id, a.shared ? 1.f / (1.f + expf(-logits[E])) : 0.f);
    }
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) last = atomicAdd(a.ticket, 1) == (int)gridDim.x - 1;
    __syncthreads();
    if (!last) return;
    __threadfence();
    if (threadIdx.x == 0) *a.ticket = 0;
    plan_tiles(a);
}

int32_t launch_route(const RouteArgs &a, int rows, int pdl, cudaStream_t st) {
    const size_t smem = sizeof(float) * kRouteWarps * (size_t)(2 * (a.experts + a.identity) + a.groups);
    JGPT_REQUIRE(smem <= 47 * 1024 && a.top <= 32, JGPT_ERR_UNSUPPORTED, "%d router outputs, %d chosen", a.experts + a.identity, a.top);
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = dim3((unsigned)((rows + kRouteWarps - 1) / kRouteWarps)), cfg.blockDim = dim3(32 * kRouteWarps), cfg.dynamicSmemBytes = smem, cfg.stream = st;
    cfg.attrs = attr, cfg.numAttrs = (pdl & 1) ? 1 : 0;
    JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, route_kernel, a, rows, pdl));
    return JGPT_OK;
}

}  // namespace mix
}  // namespace jgpt
