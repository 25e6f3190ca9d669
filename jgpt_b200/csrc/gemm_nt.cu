// C[M, N] = A[M, K] . W[N, K]^T for decode-sized M (bf16, mma.sync) and in plain fp32.
//
// Decode-sized bf16 products are bound by the weight stream and by latency: a CTA owns 32 output columns (64 from 33 rows
// on, so that the rows are read half as often) and up to 64 rows; its eight warps split every 128-wide k tile (a warp
// covers 32 columns with its own k slice), tiles arrive through a cp.async ring, and the partial tiles are added in warp
// order through shared memory.  Products with few column tiles run as clusters of CTAs that split the k range; the partial sums meet in the
// first CTA's shared memory and are added in k order: no atomics, the same bits every time.
#include "gemm_nt.cuh"

#include <algorithm>

#include "ptx.cuh"

namespace jgpt {
namespace nt {

// D(16x8, f32) += A(16x16, bf16, row) * B(16x8, bf16, col)
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

constexpr int kBK = 128, kMaxSplit = 8;

struct SmallArgs {
    Problem p[2];
    int tiles[2], per_seg[2];   // column tiles of each product, of each of its segments
    int n, k_split, pdl;
};

// Warps: NH groups of 32 columns x 8 / NH slices of the k tile.
template <int MT, int NH>
__host__ __device__ constexpr size_t small_red_bytes() { return sizeof(float) * (8 / NH) * 16 * MT * (32 * NH + 1); }
template <int MT, int NH, int STAGES>
__host__ __device__ constexpr size_t small_ring_bytes() { return (size_t)STAGES * (16 * MT + 32 * NH) * kBK * 2; }
// The ring, the reduction buffer and the other k parts' sums follow one another in the same memory.
template <int MT, int NH, int STAGES>
constexpr size_t small_smem(int k_split) {
    return std::max(std::max(small_ring_bytes<MT, NH, STAGES>(), small_red_bytes<MT, NH>()), sizeof(float) * (size_t)(k_split - 1) * 16 * MT * 32 * NH);
}

template <int MT, int NH, int STAGES, int EPI, bool GROUPED>
__global__ void __launch_bounds__(256) gemm_nt_small_kernel(const SmallArgs args) {
    constexpr int BM = 16 * MT, kBN = 32 * NH, KS = 8 / NH;
    extern __shared__ __align__(128) uint8_t nt_smem[];
    __nv_bfloat16 *As = reinterpret_cast<__nv_bfloat16 *>(nt_smem);         // [STAGES][BM][128], 16-byte chunks xor-swizzled by row
    __nv_bfloat16 *Ws = As + (size_t)STAGES * BM * kBK;                     // [STAGES][kBN][128]
    float *red = reinterpret_cast<float *>(nt_smem);                        // [KS][BM][kBN + 1], after the k loop
    float *xch = reinterpret_cast<float *>(nt_smem);                        // [k_split - 1][BM * kBN], after the reduction

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nh = warp % NH, kslice = warp / NH;
    int tile = blockIdx.x / args.k_split;
    const int k_part = blockIdx.x % args.k_split;
    const bool second = args.n > 1 && tile >= args.tiles[0];
    if (second) tile -= args.tiles[0];
    const Problem &P = second ? args.p[1] : args.p[0];
    const int N = P.N, K = P.K, lda = P.lda, ldw = P.ldw, per_seg = args.per_seg[second];
    int M = P.M, m0 = blockIdx.y * BM, seg = tile / per_seg, src0 = 0;
    bool wait = args.pdl & 1;
    const __nv_bfloat16 *__restrict__ W = reinterpret_cast<const __nv_bfloat16 *>(P.W);
    if (GROUPED) {  // a grid of one dimension: the groups' row tiles, then those of the product beside them
        if (!second) {
            if (wait && !P.grp.early) griddep_wait(), wait = false;
            if (args.pdl & 2) griddep_launch_dependents();
            if (seg >= *P.grp.n_tiles) {
                if (wait) griddep_wait();  // whoever comes next counts on this launch having waited
                return;
            }
            const RowTile t = P.grp.tiles[seg];
            m0 = t.row0, M = t.row_end, src0 = t.src0 - t.row0, W += t.group * P.grp.w_group;
        } else {
            if (args.pdl & 2) griddep_launch_dependents();
            m0 = seg * BM;
        }
        seg = 0;
    }
    const int seg_n = P.seg_n, n0 = seg * seg_n + tile % per_seg * kBN, n_end = min(N, (seg + 1) * seg_n), cn = seg * P.c_seg;
    const __nv_bfloat16 *__restrict__ A = reinterpret_cast<const __nv_bfloat16 *>(P.A) + min(seg, P.a_cap) * P.a_seg;
    const int nk_all = (K + kBK - 1) / kBK;
    const int kt0 = k_part * nk_all / args.k_split, nk = (k_part + 1) * nk_all / args.k_split - kt0;

    const int r16 = tid >> 4, c16 = tid & 15;  // chunk slot: row r16 (+ 16 i), 16-byte chunk c16 of the 128-wide tile
    auto load_w = [&](int buf, int k0) {
#pragma unroll
        for (int i = 0; i < 2 * NH; i++) {
            const int r = r16 + 16 * i, k = k0 + c16 * 8;
            const bool ok = n0 + r < n_end && k < K;
            cp_async16(Ws + ((size_t)buf * kBN + r) * kBK + ((c16 ^ (r & 7)) * 8), ok ? W + (size_t)(n0 + r) * ldw + k : W, ok);
        }
    };
    if (!GROUPED && (args.pdl & 2)) griddep_launch_dependents();
    // weights do not depend on the previous kernel: the first tiles are requested before the wait
#pragma unroll
    for (int s = 0; s < STAGES - 1; s++)
        if (s < nk) load_w(s, (kt0 + s) * kBK);
    if (wait) griddep_wait();
    const __nv_bfloat16 *a_src[MT];
    bool a_ok[MT];
#pragma unroll
    for (int i = 0; i < MT; i++) {
        const int m = m0 + r16 + 16 * i;
        a_ok[i] = m < M;
        a_src[i] = A + (size_t)(a_ok[i] ? (P.rowsel ? P.rowsel[m + src0] : m) : 0) * lda;
    }
    auto load_a = [&](int buf, int k0) {
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const int r = r16 + 16 * i, k = k0 + c16 * 8;
            const bool ok = a_ok[i] && k < K;
            cp_async16(As + ((size_t)buf * BM + r) * kBK + ((c16 ^ (r & 7)) * 8), ok ? a_src[i] + k : A, ok);
        }
    };
#pragma unroll
    for (int s = 0; s < STAGES - 1; s++) {
        if (s < nk) load_a(s, (kt0 + s) * kBK);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    float acc[MT][4][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int j = 0; j < 4; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) acc[i][j][e] = 0.f;

    for (int kt = 0; kt < nk; kt++) {
        const int buf = kt % STAGES;
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
        __syncthreads();
        if (kt + STAGES - 1 < nk) {
            const int nb = (kt + STAGES - 1) % STAGES, k0 = (kt0 + kt + STAGES - 1) * kBK;
            load_w(nb, k0);
            load_a(nb, k0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        // this warp's slice: NH k steps of 16 (chunks 2 step and 2 step + 1 of every row), columns [32 nh, + 32)
#pragma unroll
        for (int ks = 0; ks < NH; ks++) {
            const int step = kslice * NH + ks;
            uint32_t b[2][4];
#pragma unroll
            for (int h = 0; h < 2; h++) {  // 16 output columns each
                const int r = nh * 32 + h * 16 + ((lane >> 4) << 3) + (lane & 7), c = 2 * step + ((lane >> 3) & 1);
                ldmatrix_x4(b[h], Ws + ((size_t)buf * kBN + r) * kBK + ((c ^ (r & 7)) * 8));
            }
#pragma unroll
            for (int i = 0; i < MT; i++) {
                uint32_t a[4];
                const int r = i * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), c = 2 * step + (lane >> 4);
                ldmatrix_x4(a, As + ((size_t)buf * BM + r) * kBK + ((c ^ (r & 7)) * 8));
#pragma unroll
                for (int j = 0; j < 4; j++) mma_bf16(acc[i][j], a, b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // the ring is free: it becomes the reduction buffer
    {
        const int g = lane >> 2, t = lane & 3;
        float *w = red + (size_t)kslice * BM * (kBN + 1) + nh * 32;
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int j = 0; j < 4; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) w[(i * 16 + g + (e >> 1) * 8) * (kBN + 1) + j * 8 + 2 * t + (e & 1)] = acc[i][j][e];
    }
    __syncthreads();
    constexpr int PER = BM * kBN / 256;
    float sum[PER];
#pragma unroll
    for (int i = 0; i < PER; i++) {
        const int e = tid + 256 * i;
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < KS; w++) s += red[(size_t)w * BM * (kBN + 1) + e / kBN * (kBN + 1) + e % kBN];
        sum[i] = s;
    }
    if (args.k_split > 1) {
        cluster_sync();  // every CTA of the cluster is past its reduction: its shared memory may be written
        if (k_part > 0) {
#pragma unroll
            for (int i = 0; i < PER; i++) st_cluster_f32(&xch[(size_t)(k_part - 1) * BM * kBN + tid + 256 * i], 0, sum[i]);
        }
        cluster_sync();
        if (k_part > 0) return;
        for (int s = 0; s + 1 < args.k_split; s++)
#pragma unroll
            for (int i = 0; i < PER; i++) sum[i] += xch[(size_t)s * BM * kBN + tid + 256 * i];
    }
#pragma unroll
    for (int i = 0; i < PER; i++) {
        const int e = tid + 256 * i, m = m0 + e / kBN, c = e % kBN, n = n0 + c;
        if (EPI == EPI_GATE) {
            // lanes 0-15 of a warp hold the gate of a row's 16 outputs, lanes 16-31 the linear part
            const float up = __shfl_down_sync(0xffffffffu, sum[i], 16);
            if ((c & 31) < 16 && m < M && n + 16 < N)
                reinterpret_cast<__nv_bfloat16 *>(P.C)[(size_t)m * P.ldc + n / 32 * 16 + (c & 15)] = __float2bfloat16(activate<true>(P.act, 0.f, 0.f, sum[i]) * up);
        } else if (m < M && n < n_end) {
            const size_t at = (size_t)m * P.ldc + n + cn;
            if (EPI == EPI_STORE) reinterpret_cast<__nv_bfloat16 *>(P.C)[at] = __float2bfloat16(P.bias ? sum[i] + P.bias[n] : sum[i]);
            if (EPI == EPI_ACT) reinterpret_cast<__nv_bfloat16 *>(P.C)[at] = __float2bfloat16(activate<true>(P.act, P.p0, P.p1, sum[i]));
            if (EPI == EPI_ACT_SOME)
                reinterpret_cast<__nv_bfloat16 *>(P.C)[at] = __float2bfloat16(n >= P.act_from && n < P.act_to ? activate<true>(P.act, P.p0, P.p1, sum[i]) : sum[i] + P.bias[n]);
            if (EPI == EPI_ADD_F32) reinterpret_cast<float *>(P.C)[at] = P.res_scale * P.res[at] + (P.colscale ? P.colscale[n] * sum[i] : sum[i]);
            if (EPI == EPI_SCALE_F32) reinterpret_cast<float *>(P.C)[at] = sum[i] * P.scale;
        }
    }
}

template <int MT, int NH, int STAGES, int EPI, bool GROUPED>
static int32_t small_launch(const SmallArgs &args, int total_tiles, int M, cudaStream_t st) {
    auto kern = gemm_nt_small_kernel<MT, NH, STAGES, EPI, GROUPED>;
    const size_t smem = small_smem<MT, NH, STAGES>(args.k_split);
    static thread_local int set_for = -1;  // the opt-in to more than 48 KiB, once per device
    int dev = 0;
    JGPT_CUDA_TRY(cudaGetDevice(&dev));
    if (set_for != dev) {
        JGPT_CUDA_TRY(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(small_smem<MT, NH, STAGES>(kMaxSplit))));
        set_for = dev;
    }
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[2];
    int na = 0;
    if (args.k_split > 1) {
        attr[na].id = cudaLaunchAttributeClusterDimension;
        attr[na].val.clusterDim.x = (unsigned)args.k_split, attr[na].val.clusterDim.y = 1, attr[na].val.clusterDim.z = 1;
        na++;
    }
    if (args.pdl & 1) {
        attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[na].val.programmaticStreamSerializationAllowed = 1;
        na++;
    }
    cfg.gridDim = dim3((unsigned)(total_tiles * args.k_split), GROUPED ? 1u : (unsigned)((M + 16 * MT - 1) / (16 * MT)));
    cfg.blockDim = dim3(256), cfg.dynamicSmemBytes = smem, cfg.stream = st, cfg.attrs = attr, cfg.numAttrs = (unsigned)na;
    JGPT_CUDA_TRY(cudaLaunchKernelEx(&cfg, kern, args));
    return JGPT_OK;
}

template <int EPI, bool GROUPED = false>
static int32_t small_dispatch(const Ctx *ctx, const Problem *p, int n, int pdl, cudaStream_t st) {
    SmallArgs a{};
    a.n = n, a.pdl = pdl;
    const int M = p[0].M;
    // few columns (a router's): lower tiles, so that the launch has more CTAs
    const int tall = GROUPED ? p[0].grp.rows : (n == 1 && p[0].N <= 256 ? std::min(M, 32) : M);
    const int mt = tall <= 16 ? 1 : (tall <= 32 ? 2 : 4), bn = mt == 4 ? 64 : 32, max_split = mt == 4 ? 4 : kMaxSplit;
    int tiles = 0, K = 0;
    for (int i = 0; i < n; i++) {
        a.p[i] = p[i];
        a.per_seg[i] = (p[i].seg_n + bn - 1) / bn, a.tiles[i] = p[i].column_tiles(bn);
        if (GROUPED) a.tiles[i] *= i == 0 ? p[0].grp.max_tiles : (M + 16 * mt - 1) / (16 * mt);
        tiles += a.tiles[i];
        K = std::max(K, p[i].K);
    }
    const int ctas = tiles * ((M + 16 * mt - 1) / (16 * mt)), nk = (K + kBK - 1) / kBK;
    // split k while the launch leaves SMs idle and every part keeps two tiles
    a.k_split = 1;
    while (n == 1 && !GROUPED && a.k_split < max_split && ctas * a.k_split * 2 <= 2 * ctx->sm_count && nk / (a.k_split * 2) >= 2) a.k_split *= 2;
    switch (mt) {
        case 1: return small_launch<1, 1, 6, EPI, GROUPED>(a, tiles, M, st);
        case 2: return small_launch<2, 1, 5, EPI, GROUPED>(a, tiles, M, st);
        default: return small_launch<4, 2, 3, EPI, GROUPED>(a, tiles, M, st);
    }
}

int umma_min_rows() {
    static const int v = env_int("JGPT_B200_NT_UMMA_MIN_ROWS", 129);
    return v;
}

int group_tile_rows(bool f32, int rows, int copies, int groups) {
    if (f32) return 64;
    if (umma_min_rows() > 0 && rows >= umma_min_rows()) return kLargeTile;
    const int mean = (rows * copies + groups - 1) / groups;
    return mean <= 10 ? 16 : (mean <= 22 ? 32 : 64);
}

// Defaults spelled out: one segment, the residual in C itself.
static int32_t complete(const Problem *p, int n, Epilogue epi, Problem (&q)[2]) {
    JGPT_REQUIRE(n >= 1 && n <= 2 && p[0].M > 0, JGPT_ERR_INVALID_ARGUMENT, "1 or 2 products per launch");
    for (int i = 0; i < n; i++) {
        q[i] = p[i];
        if (q[i].seg_n <= 0) q[i].seg_n = q[i].N;
        if (!q[i].res) q[i].res = reinterpret_cast<const float *>(q[i].C);
        JGPT_REQUIRE(epi != EPI_ACT_SOME || q[i].bias, JGPT_ERR_INVALID_ARGUMENT, "columns without an activation need a bias");
        JGPT_REQUIRE(!q[i].grp.tiles || (i == 0 && (epi == EPI_STORE || epi == EPI_ACT) && q[i].segments() == 1 && q[i].grp.max_tiles > 0),
                     JGPT_ERR_INVALID_ARGUMENT, "rows in groups: the first product of a launch, one segment, stored or activated");
    }
    return JGPT_OK;
}

int32_t launch_bf16(const Ctx *ctx, const Problem *problems, int n, Epilogue epi, int pdl, cudaStream_t st) {
    Problem p[2];
    if (int32_t rc = complete(problems, n, epi, p)) return rc;
    bool big = p[0].M >= umma_min_rows() && umma_min_rows() > 0;
    for (int i = 0; i < n; i++) big = big && !p[i].rowsel;
    if (p[0].grp.tiles) {
        const int rows = p[0].grp.rows;
        JGPT_REQUIRE(big ? rows == kLargeTile : (rows == 16 || rows == 32 || rows == 64), JGPT_ERR_INVALID_ARGUMENT, "row tiles of %d", rows);
        if (!big) return epi == EPI_ACT ? small_dispatch<EPI_ACT, true>(ctx, p, n, pdl, st) : small_dispatch<EPI_STORE, true>(ctx, p, n, pdl, st);
    }
    if (big) {
        for (int i = 0; i < n; i++)
            if (int32_t rc = launch_bf16_umma(ctx, p[i], epi, pdl, st)) return rc;
        return JGPT_OK;
    }
    switch (epi) {
        case EPI_STORE: return small_dispatch<EPI_STORE>(ctx, p, n, pdl, st);
        case EPI_ADD_F32: return small_dispatch<EPI_ADD_F32>(ctx, p, n, pdl, st);
        case EPI_SCALE_F32: return small_dispatch<EPI_SCALE_F32>(ctx, p, n, pdl, st);
        case EPI_GATE: return small_dispatch<EPI_GATE>(ctx, p, n, pdl, st);
        case EPI_ACT: return small_dispatch<EPI_ACT>(ctx, p, n, pdl, st);
        case EPI_ACT_SOME: return small_dispatch<EPI_ACT_SOME>(ctx, p, n, pdl, st);
    }
    return fail(JGPT_ERR_INVALID_ARGUMENT, "unknown epilogue");
}

// ------------------------------------------------------------------------------------------------
// Plain fp32: 64 x 64 tiles, fused multiply-add, k in ascending order in one thread.  The exact mode of the forward step.
// ------------------------------------------------------------------------------------------------
template <int EPI>
__global__ void __launch_bounds__(256) gemm_nt_f32_kernel(const Problem P0, const Problem P1) {
    constexpr int BT = 64, BK = 16;
    __shared__ float As[BK][BT + 1], Ws[BK][BT + 1];
    const Problem &P = blockIdx.z == 0 ? P0 : P1;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int per_seg = (P.seg_n + BT - 1) / BT, seg = blockIdx.x / per_seg, cn = seg * P.c_seg;
    const int n0 = seg * P.seg_n + blockIdx.x % per_seg * BT, n_end = min(P.N, (seg + 1) * P.seg_n);
    if (n0 >= P.N) return;
    const float *__restrict__ A = reinterpret_cast<const float *>(P.A) + min(seg, P.a_cap) * P.a_seg;
    const float *__restrict__ W = reinterpret_cast<const float *>(P.W);
    int m0 = blockIdx.y * BT, m_end = P.M, src0 = 0;
    if (P.grp.tiles) {
        if ((int)blockIdx.y >= *P.grp.n_tiles) return;
        const RowTile t = P.grp.tiles[blockIdx.y];
        m0 = t.row0, m_end = t.row_end, src0 = t.src0 - t.row0, W += t.group * P.grp.w_group;
    }
    float acc[4][4] = {};
    for (int k0 = 0; k0 < P.K; k0 += BK) {
        for (int e = tid; e < BT * BK; e += 256) {
            const int r = e / BK, k = k0 + e % BK, m = m0 + r, n = n0 + r;
            As[e % BK][r] = (m < m_end && k < P.K) ? A[(size_t)(P.rowsel ? P.rowsel[m + src0] : m) * P.lda + k] : 0.f;
            Ws[e % BK][r] = (n < n_end && k < P.K) ? W[(size_t)n * P.ldw + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < BK; kk++) {
            float a[4], w[4];
#pragma unroll
            for (int i = 0; i < 4; i++) a[i] = As[kk][ty * 4 + i], w[i] = Ws[kk][tx + 16 * i];
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
        }
        __syncthreads();
    }
    float *C = reinterpret_cast<float *>(P.C);
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int m = m0 + ty * 4 + i;
        if (m >= m_end) continue;
        if (EPI == EPI_GATE) {  // columns tx (+ 32) of a group of 32 are the gate, tx + 16 the linear part
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int n = n0 + tx + 16 * j;
                if (n + 16 < P.N) C[(size_t)m * P.ldc + n / 32 * 16 + tx] = activate<false>(P.act, 0.f, 0.f, acc[i][j]) * acc[i][j + 1];
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int n = n0 + tx + 16 * j;
                if (n >= n_end) continue;
                const size_t at = (size_t)m * P.ldc + n + cn;
                if (EPI == EPI_STORE) C[at] = P.bias ? acc[i][j] + P.bias[n] : acc[i][j];
                if (EPI == EPI_ACT) C[at] = activate<false>(P.act, P.p0, P.p1, acc[i][j]);
                if (EPI == EPI_ACT_SOME) C[at] = n >= P.act_from && n < P.act_to ? activate<false>(P.act, P.p0, P.p1, acc[i][j]) : acc[i][j] + P.bias[n];
                if (EPI == EPI_ADD_F32) C[at] = P.res_scale * P.res[at] + (P.colscale ? P.colscale[n] * acc[i][j] : acc[i][j]);
                if (EPI == EPI_SCALE_F32) C[at] = acc[i][j] * P.scale;
            }
        }
    }
}

int32_t launch_f32(const Problem *problems, int n, Epilogue epi, cudaStream_t st) {
    Problem p[2];
    if (int32_t rc = complete(problems, n, epi, p)) return rc;
    const Problem &q = p[n - 1];
    if (p[0].grp.tiles && n == 2) {
        if (int32_t rc = launch_f32(p, 1, epi, st)) return rc;
        return launch_f32(p + 1, 1, epi, st);
    }
    JGPT_REQUIRE(!p[0].grp.tiles || p[0].grp.rows <= 64, JGPT_ERR_INVALID_ARGUMENT, "row tiles of %d", p[0].grp.rows);
    auto tiles = [](const Problem &x) { return x.column_tiles(64); };
    const dim3 grid((unsigned)std::max(tiles(p[0]), tiles(q)), (unsigned)(p[0].grp.tiles ? p[0].grp.max_tiles : (p[0].M + 63) / 64), (unsigned)n);
    switch (epi) {
        case EPI_STORE: gemm_nt_f32_kernel<EPI_STORE><<<grid, 256, 0, st>>>(p[0], q); break;
        case EPI_ADD_F32: gemm_nt_f32_kernel<EPI_ADD_F32><<<grid, 256, 0, st>>>(p[0], q); break;
        case EPI_SCALE_F32: gemm_nt_f32_kernel<EPI_SCALE_F32><<<grid, 256, 0, st>>>(p[0], q); break;
        case EPI_GATE: gemm_nt_f32_kernel<EPI_GATE><<<grid, 256, 0, st>>>(p[0], q); break;
        case EPI_ACT: gemm_nt_f32_kernel<EPI_ACT><<<grid, 256, 0, st>>>(p[0], q); break;
        case EPI_ACT_SOME: gemm_nt_f32_kernel<EPI_ACT_SOME><<<grid, 256, 0, st>>>(p[0], q); break;
    }
    JGPT_CUDA_TRY(cudaGetLastError());
    return JGPT_OK;
}

}  // namespace nt
}  // namespace jgpt
