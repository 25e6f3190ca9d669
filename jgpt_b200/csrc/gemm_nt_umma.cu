// C[M, N] = A[M, K] . W[N, K]^T for prefill-sized M on the 5th-generation tensor cores: tcgen05.mma kind::f16 over bf16
// operands, fp32 accumulator double-buffered in tensor memory.
//
// Both operands are row major with K contiguous, so TMA tensor maps bring 64-wide k tiles into shared memory in the
// 128-byte swizzled K-major layout the tensor core reads: row r of a tile at r * 128 bytes, its 16-byte chunks permuted
// by r % 8; eight-row groups 1024 bytes apart (the descriptor's stride offset); one 16-wide k step advances the start
// address by 32 bytes.  Rows and columns past the operands read as zeros, so no shape needs padding beyond 16-byte rows.
//
// Persistent CTAs of 320 threads: warp 0 issues the copies, warp 1 owns the tensor memory and issues the MMAs, warps 2-9
// drain the accumulator (TMEM lane quarter = warp % 4, half the tile's columns each) while the next tile is multiplied.
// Rows in groups (experts): the device's list of row tiles takes the place of the row grid and the weight tile's rows
// shift by group.
// Output tiles are walked in groups of eight row tiles, rows fastest, so CTAs side by side share weight tiles in L2.
// Every wait is bounded; on expiry the status word gets DEV_STATUS_WAIT_TIMEOUT and the CTA winds down.
#include <cuda.h>

#include <algorithm>

#include "gemm_nt.cuh"
#include "tcgen05.cuh"

namespace jgpt {
namespace nt {

constexpr int UM = 128, UK = 64, kEpiWarps = 8, kUmmaThreads = 64 + 32 * kEpiWarps, kGroupM = 8;
template <int BN>
__host__ __device__ constexpr uint32_t stage_bytes() { return (UM + BN) * UK * 2; }
template <int BN>
__host__ __device__ constexpr int stages() { return BN == 256 ? 4 : (BN == 128 ? 6 : 8); }
template <int BN>
__host__ __device__ constexpr uint32_t umma_smem() { return stages<BN>() * stage_bytes<BN>() + 1024; }

// K-major operand with 128-byte swizzle: start address, stride offset 1024, version 1 (bits 46-47), layout 2 (bits 61-63).
__device__ __forceinline__ uint64_t desc_sw128(uint32_t saddr) {
    return (uint64_t)((saddr & 0x3FFFFu) >> 4) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void mma_bf16_ss(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}
__device__ __forceinline__ void tma_2d(void *smem_dst, const CUtensorMap *map, int x, int y, uint64_t *bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(
                     smem_u32(smem_dst)),
                 "l"(map), "r"(x), "r"(y), "r"(smem_u32(bar))
                 : "memory");
}

enum RowMode : int { ROWS_ALL = 0, ROWS_GROUPS = 1 };

struct UmmaArgs {
    void *C;
    int M, N, K, ldc, mt, nt, pdl;
    float scale;
    int *status;
    int per_seg, seg_n, c_seg, a_x, a_y, a_cap;  // column tiles and columns of a segment; its shift in C; its operand's shift (columns, rows), up to a_cap times
    const float *res, *colscale, *bias;
    int act, act_from, act_to;
    float p0, p1, res_scale;
    const RowTile *tiles;  // groups: the row tiles, how many, each group's rows of W
    const int *n_tiles;
    int w_rows;
};

__device__ __forceinline__ void tile_of(const UmmaArgs &a, int mt, int t, int &m, int &n) {
    const int per = kGroupM * a.nt, g = t / per, r = t % per, gm = min(kGroupM, mt - g * kGroupM);
    m = g * kGroupM + r % gm, n = r / gm;
}

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t *>(&v);
}

// bias: of v[0], on a 16-byte boundary; of n columns.
__device__ __forceinline__ void add_bias(float (&v)[32], const float *bias, int n) {
#pragma unroll
    for (int q = 0; q < 32; q += 4)
        if (q < n) {  // multiples of 8 here
            const float4 b = __ldg(reinterpret_cast<const float4 *>(bias + q));
            v[q] += b.x, v[q + 1] += b.y, v[q + 2] += b.z, v[q + 3] += b.w;
        }
}

template <int BN, int EPI, int ROWS>
__global__ void __launch_bounds__(kUmmaThreads, 1) gemm_nt_umma_kernel(const __grid_constant__ CUtensorMap amap, const __grid_constant__ CUtensorMap wmap,
                                                                       const UmmaArgs a) {
    constexpr int ST = stages<BN>();
    constexpr uint32_t SB = stage_bytes<BN>(), A_BYTES = UM * UK * 2, COLS = 2 * BN;
    constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(UM >> 4) << 24);
    extern __shared__ uint8_t umma_raw[];
    __shared__ __align__(8) uint64_t full_bar[ST], empty_bar[ST], acc_full[2], acc_empty[2];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort_mem;
    volatile int *s_abort = &s_abort_mem;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nk = (a.K + UK - 1) / UK;
    uint8_t *tiles = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(umma_raw) + 1023) & ~(uintptr_t)1023);

    if (tid == 0) {
        for (int s = 0; s < ST; s++) mbar_init(&full_bar[s], 1), mbar_init(&empty_bar[s], 1);
        for (int b = 0; b < 2; b++) mbar_init(&acc_full[b], 1), mbar_init(&acc_empty[b], kEpiWarps);
        *s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(&s_tmem, COLS);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    if (a.pdl & 2) griddep_launch_dependents();
    if (a.pdl & 1) griddep_wait();
    const int mt = ROWS == ROWS_ALL ? a.mt : min(*a.n_tiles, a.mt), total = mt * a.nt;

    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;
            for (int t = blockIdx.x; t < total && !*s_abort; t += gridDim.x) {
                int m, n;
                tile_of(a, mt, t, m, n);
                const int seg = n / a.per_seg, shift = min(seg, a.a_cap), ax = shift * a.a_x;
                int ay = shift * a.a_y + m * UM, wy = seg * a.seg_n + n % a.per_seg * BN;
                if (ROWS != ROWS_ALL) ay = a.tiles[m].row0, wy += a.tiles[m].group * a.w_rows;
                for (int kt = 0; kt < nk; kt++, it++) {
                    const uint32_t s = it % ST, use = it / ST;
                    if (use > 0 && !mbar_wait_bounded(&empty_bar[s], (use - 1) & 1u, a.status, s_abort)) break;
                    uint8_t *dst = tiles + (size_t)s * SB;
                    mbar_expect_tx(&full_bar[s], SB);
                    tma_2d(dst, &amap, ax + kt * UK, ay, &full_bar[s]);
                    tma_2d(dst + A_BYTES, &wmap, kt * UK, wy, &full_bar[s]);
                }
            }
            if (*s_abort) {  // copies already issued still target this CTA's shared memory: give each a bounded chance to land
                for (uint32_t k = it > (uint32_t)ST ? it - ST : 0; k < it; k++)
                    for (uint32_t i = 0; i < (1u << 16) && !mbar_try_wait(&full_bar[k % ST], (k / ST) & 1u); i++) {
                    }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            uint32_t it = 0, j = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < total && ok; t += gridDim.x, j++) {
                const uint32_t buf = j & 1u, round = j >> 1;
                if (round > 0 && !mbar_wait_bounded(&acc_empty[buf], (round - 1) & 1u, a.status, s_abort)) break;
                tc_fence_after();
                const uint32_t acc = tmem + buf * BN;
                for (int kt = 0; kt < nk; kt++, it++) {
                    const uint32_t s = it % ST, use = it / ST;
                    if (!mbar_wait_bounded(&full_bar[s], use & 1u, a.status, s_abort)) {
                        ok = false;
                        break;
                    }
                    tc_fence_after();
                    const uint32_t sa = smem_u32(tiles + (size_t)s * SB), sw = sa + A_BYTES;
#pragma unroll
                    for (int ks = 0; ks < UK / 16; ks++) mma_bf16_ss(acc, desc_sw128(sa + ks * 32), desc_sw128(sw + ks * 32), IDESC, (kt | ks) != 0);
                    mma_commit(&empty_bar[s]);
                }
                if (ok) mma_commit(&acc_full[buf]);
            }
        }
    } else {
        const int quarter = warp & 3, half = (warp - 2) >> 2;
        const bool vec4 = (a.ldc & 3) == 0 && (a.c_seg & 3) == 0;
        uint32_t j = 0;
        for (int t = blockIdx.x; t < total; t += gridDim.x, j++) {
            const uint32_t buf = j & 1u, round = j >> 1, acc = tmem + buf * BN;
            int mi, ni;
            tile_of(a, mt, t, mi, ni);
            const int row0 = ROWS == ROWS_ALL ? mi * UM : a.tiles[mi].row0, m_end = ROWS == ROWS_ALL ? a.M : a.tiles[mi].row_end;
            const int seg = ni / a.per_seg, m = row0 + quarter * 32 + lane, n0 = seg * a.seg_n + ni % a.per_seg * BN;
            const int n_end = min(a.N, (seg + 1) * a.seg_n), cn = seg * a.c_seg;
            int ok = 0;
            if (lane == 0) ok = mbar_wait_bounded(&acc_full[buf], round & 1u, a.status, s_abort) ? 1 : 0;
            ok = __shfl_sync(0xffffffffu, ok, 0);
            if (!ok) break;
            tc_fence_after();
#pragma unroll 1
            for (int c0 = half * (BN / 2); c0 < (half + 1) * (BN / 2); c0 += 32) {
                if (n0 + c0 >= n_end) break;  // uniform across the warp
                float v[32];
                load_acc32(acc, quarter, c0, v);
                if (m >= m_end) continue;
                if (EPI == EPI_STORE || EPI == EPI_ACT || EPI == EPI_ACT_SOME) {
                    __nv_bfloat16 *c = reinterpret_cast<__nv_bfloat16 *>(a.C) + (size_t)m * a.ldc + n0 + c0 + cn;
                    const int n1 = n0 + c0;
                    if (EPI == EPI_ACT_SOME) {
                        if (n1 >= a.act_to || n1 + 32 <= a.act_from) {
                            add_bias(v, a.bias + n1, n_end - n1);
                        } else if (n1 >= a.act_from && n1 + 32 <= a.act_to && a.act == ACT_RELU2) {
#pragma unroll
                            for (int q = 0; q < 32; q++) v[q] = fmaxf(v[q], 0.f), v[q] *= v[q];
                        } else {
                            float w[32];
#pragma unroll
                            for (int q = 0; q < 32; q++) w[q] = activate<true>(a.act, a.p0, a.p1, v[q]);
                            add_bias(v, a.bias + n1, n_end - n1);
#pragma unroll
                            for (int q = 0; q < 32; q++)
                                if (n1 + q >= a.act_from && n1 + q < a.act_to) v[q] = w[q];
                        }
                    } else if (EPI == EPI_ACT && a.act == ACT_XIELU) {
#pragma unroll
                        for (int q = 0; q < 32; q++) v[q] = xielu_fast(v[q], a.p0, a.p1);
                    } else if (EPI == EPI_ACT && a.act == ACT_TANH) {
#pragma unroll
                        for (int q = 0; q < 32; q++) v[q] = tanhf(v[q]);
                    } else if (EPI == EPI_ACT && a.act == ACT_RELU2) {
#pragma unroll
                        for (int q = 0; q < 32; q++) v[q] = fmaxf(v[q], 0.f), v[q] *= v[q];
                    } else if (EPI == EPI_ACT) {
#pragma unroll
                        for (int q = 0; q < 32; q++) v[q] = activate<true>(a.act, a.p0, a.p1, v[q]);
                    }
                    if (EPI == EPI_STORE && a.bias) add_bias(v, a.bias + n1, n_end - n1);
#pragma unroll
                    for (int q = 0; q < 4; q++)
                        if (n0 + c0 + 8 * q < n_end)  // N and seg_n are multiples of 8 here
                            *reinterpret_cast<uint4 *>(c + 8 * q) = make_uint4(pack_bf16(v[8 * q], v[8 * q + 1]), pack_bf16(v[8 * q + 2], v[8 * q + 3]),
                                                                               pack_bf16(v[8 * q + 4], v[8 * q + 5]), pack_bf16(v[8 * q + 6], v[8 * q + 7]));
                } else if (EPI == EPI_GATE) {
                    __nv_bfloat16 *c = reinterpret_cast<__nv_bfloat16 *>(a.C) + (size_t)m * a.ldc + (n0 + c0) / 2;
                    if (a.act == ACT_RELU) {
#pragma unroll
                        for (int q = 0; q < 16; q++) v[q] = fmaxf(v[q], 0.f) * v[16 + q];
                    } else {
#pragma unroll
                        for (int q = 0; q < 16; q++) v[q] = gelu_tanh(v[q]) * v[16 + q];
                    }
#pragma unroll
                    for (int q = 0; q < 2; q++)
                        *reinterpret_cast<uint4 *>(c + 8 * q) = make_uint4(pack_bf16(v[8 * q], v[8 * q + 1]), pack_bf16(v[8 * q + 2], v[8 * q + 3]),
                                                                           pack_bf16(v[8 * q + 4], v[8 * q + 5]), pack_bf16(v[8 * q + 6], v[8 * q + 7]));
                } else {
                    const size_t at = (size_t)m * a.ldc + n0 + c0 + cn;
                    float *c = reinterpret_cast<float *>(a.C) + at;
                    const float *res = a.res + at;
                    if (EPI == EPI_ADD_F32 && a.colscale) {
#pragma unroll
                        for (int q = 0; q < 32; q++)
                            if (n0 + c0 + q < n_end) v[q] *= __ldg(a.colscale + n0 + c0 + q);
                    }
#pragma unroll
                    for (int q = 0; q < 8; q++) {
                        const int n = n0 + c0 + 4 * q;
                        float4 o = make_float4(v[4 * q], v[4 * q + 1], v[4 * q + 2], v[4 * q + 3]);
                        if (EPI == EPI_SCALE_F32) o.x *= a.scale, o.y *= a.scale, o.z *= a.scale, o.w *= a.scale;
                        if (vec4 && n + 3 < n_end) {
                            if (EPI == EPI_ADD_F32) {
                                const float4 r = *reinterpret_cast<const float4 *>(res + 4 * q);
                                o.x = fmaf(a.res_scale, r.x, o.x), o.y = fmaf(a.res_scale, r.y, o.y), o.z = fmaf(a.res_scale, r.z, o.z), o.w = fmaf(a.res_scale, r.w, o.w);
                            }
                            *reinterpret_cast<float4 *>(c + 4 * q) = o;
                        } else {
                            const float e[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
                            for (int i = 0; i < 4; i++)
                                if (n + i < n_end) c[4 * q + i] = EPI == EPI_ADD_F32 ? fmaf(a.res_scale, res[4 * q + i], e[i]) : e[i];
                        }
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[buf]);
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem, COLS);
    }
}

typedef CUresult (*EncodeFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *,
                             const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static EncodeFn encode_fn() {
    static EncodeFn fn = [] {
        void *p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) p = nullptr;
        return reinterpret_cast<EncodeFn>(p);
    }();
    return fn;
}
// [rows, K] bf16, row stride ld elements, boxes of 64 x box_rows.
static int32_t make_map(CUtensorMap *map, const void *base, int rows, int K, int ld, int box_rows) {
    EncodeFn fn = encode_fn();
    JGPT_REQUIRE(fn, JGPT_ERR_CUDA, "the driver has no cuTensorMapEncodeTiled");
    const cuuint64_t dims[2] = {(cuuint64_t)K, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {UK, (cuuint32_t)box_rows}, elem[2] = {1, 1};
    const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                          CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    JGPT_REQUIRE(r == CUDA_SUCCESS, JGPT_ERR_CUDA, "tensor map of [%d, %d] stride %d refused (%d)", rows, K, ld, (int)r);
    return JGPT_OK;
}

template <int BN, int EPI, int ROWS>
static int32_t umma_launch(const Ctx *ctx, const Problem &p, int pdl, cudaStream_t st) {
    CUtensorMap am, wm;
    const int segs = p.segments(), shifts = std::min(segs - 1, p.a_cap), ay = (int)(p.a_seg / p.lda), ax = (int)(p.a_seg % p.lda), per_seg = (p.segment_cols() + BN - 1) / BN;
    const int w_rows = ROWS == ROWS_ALL ? 0 : (int)(p.grp.w_group / p.ldw), mt = ROWS == ROWS_ALL ? (p.M + UM - 1) / UM : p.grp.max_tiles;
    int32_t rc = make_map(&am, p.A, ROWS == ROWS_ALL ? p.M + shifts * ay : p.grp.a_rows, p.K + shifts * ax, p.lda, UM);
    if (!rc) rc = make_map(&wm, p.W, ROWS == ROWS_ALL ? p.N : (p.grp.n_groups - 1) * w_rows + p.N, p.K, p.ldw, BN);
    if (rc) return rc;
    UmmaArgs a{p.C, p.M, p.N, p.K, p.ldc, mt, p.column_tiles(BN), pdl, p.scale, ctx->d_status,
               per_seg, p.segment_cols(), p.c_seg, ax, ay, p.a_cap, p.res, p.colscale, p.bias, p.act, p.act_from, p.act_to, p.p0, p.p1, p.res_scale,
               p.grp.tiles, p.grp.n_tiles, w_rows};
    auto kern = gemm_nt_umma_kernel<BN, EPI, ROWS>;
    static thread_local int set_for = -1;
    if (set_for != ctx->device) {
        JGPT_CUDA_TRY(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)umma_smem<BN>()));
        set_for = ctx->device;
    }
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = dim3((unsigned)std::min(a.mt * a.nt, ctx->sm_count)), cfg.blockDim = dim3(kUmmaThreads);
    cfg.dynamicSmemBytes = umma_smem<BN>(), cfg.stream = st, cfg.attrs = attr, cfg.numAttrs = (pdl & 1) ? 1 : 0;
    JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, kern, (const CUtensorMap)am, (const CUtensorMap)wm, (const UmmaArgs)a));
    return JGPT_OK;
}

template <int EPI, int ROWS = ROWS_ALL>
static int32_t umma_pick(const Ctx *ctx, const Problem &p, int pdl, cudaStream_t st) {
    const int mt = ROWS == ROWS_ALL ? (p.M + UM - 1) / UM : p.grp.max_tiles;
    auto tiles = [&](int bn) { return mt * p.column_tiles(bn); };
    if (tiles(256) >= ctx->sm_count) return umma_launch<256, EPI, ROWS>(ctx, p, pdl, st);
    if (tiles(128) >= ctx->sm_count * 2 / 3) return umma_launch<128, EPI, ROWS>(ctx, p, pdl, st);
    return umma_launch<64, EPI, ROWS>(ctx, p, pdl, st);
}

int32_t launch_bf16_umma(const Ctx *ctx, const Problem &p, Epilogue epi, int pdl, cudaStream_t st) {
    JGPT_REQUIRE(p.lda % 8 == 0 && p.ldw % 8 == 0 && (reinterpret_cast<uintptr_t>(p.A) & 15) == 0 && (reinterpret_cast<uintptr_t>(p.W) & 15) == 0,
                 JGPT_ERR_INVALID_ARGUMENT, "operand rows must start on 16-byte boundaries");
    JGPT_REQUIRE((epi != EPI_STORE || (p.N % 8 == 0 && p.ldc % 8 == 0)) && (epi != EPI_GATE || ((p.act == ACT_GELU || p.act == ACT_RELU) && p.N % 32 == 0 && p.ldc % 8 == 0)),
                 JGPT_ERR_INVALID_ARGUMENT, "output columns %d, stride %d", p.N, p.ldc);
    JGPT_REQUIRE(((epi != EPI_ACT && epi != EPI_ACT_SOME) || (p.N % 8 == 0 && p.ldc % 8 == 0)) &&
                     (p.segments() == 1 || (p.seg_n % 8 == 0 && p.c_seg % 8 == 0 && p.a_seg % 8 == 0 && epi != EPI_GATE)),
                 JGPT_ERR_INVALID_ARGUMENT, "segments of %d columns, shifts %lld / %d", p.seg_n, p.a_seg, p.c_seg);
    if (p.grp.tiles) {
        JGPT_REQUIRE(p.grp.n_groups > 0 && p.grp.a_rows > 0 && p.grp.w_group % p.ldw == 0, JGPT_ERR_INVALID_ARGUMENT, "groups of rows");
        return epi == EPI_ACT ? umma_pick<EPI_ACT, ROWS_GROUPS>(ctx, p, pdl, st) : umma_pick<EPI_STORE, ROWS_GROUPS>(ctx, p, pdl, st);
    }
    switch (epi) {
        case EPI_ACT: return umma_pick<EPI_ACT>(ctx, p, pdl, st);
        case EPI_ACT_SOME: return umma_pick<EPI_ACT_SOME>(ctx, p, pdl, st);
        case EPI_STORE: return umma_pick<EPI_STORE>(ctx, p, pdl, st);
        case EPI_ADD_F32: return umma_pick<EPI_ADD_F32>(ctx, p, pdl, st);
        case EPI_SCALE_F32: return umma_pick<EPI_SCALE_F32>(ctx, p, pdl, st);
        case EPI_GATE: return umma_pick<EPI_GATE>(ctx, p, pdl, st);
    }
    return fail(JGPT_ERR_INVALID_ARGUMENT, "unknown epilogue");
}

}  // namespace nt
}  // namespace jgpt
