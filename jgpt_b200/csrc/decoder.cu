// Layered decoder: configuration, weights, step function.
//
// A layer is  x <- x + sum of its mixer branches(LN1(x)),  then  x <- x + ff(LN2(x))  when it has a feed-forward part (norms may
// come behind the sums instead, see below).
// All branches of a layer read the same normalised rows, so their input projections are ONE product over concatenated
// weights, and their output projections are ONE product over concatenated (gated, scaled) head outputs that adds to the
// residual in its epilogue:
//
//   LN1 -> proj = h W_in^T -> [z = low-rank second factors] -> mixer kernels -> x += mixed W_out^T -> LN2 -> gelu pair -> x += act W_down^T
//
// With RMS norms the residual may be an average over the depth: every layer's result stays in a slot of its own, the norm in front of the
// next layer forms the weighted sum on its way, and the product epilogues add (times the layer scale) to the slot.  A WKV layer's
// norm writes five mixes with the previous token's row, which its input projections read as segments of one product.
//
// With norms behind the sums the parts read x itself: the product epilogues form residual factor x x + part, the norm kernel
// behind them writes x and its rounding for the next product.  A mixture of experts is router -> route (choice, lists, tiles) ->
// up products of all experts and the shared one -> down products -> the norm kernel adds a token's weighted rows on its way.
//
// With norms on both sides of the parts the norm kernel between two parts does everything but products: it gates and norms the part's
// result, adds it to x (two arrays in turn), norms x for the next part and mixes in the row before.  The gate's projection rides
// with the next part's first product: a second segment of it reads the rows as they were before the shift.
//
// The residual x is fp32; rows entering a product are bf16 (or fp32 in the exact mode).  Head sizes are padded with zero
// weights to what the kernels take, so every size of a configuration works; sums over a head use the true size.
#include "decoder.cuh"

#include <algorithm>
#include <cmath>
#include <memory>

#include "gemm_nt.cuh"
#include "mixers.cuh"

namespace jgpt {

static int up(int n, int m) { return (n + m - 1) / m * m; }

struct DBranch {
    jgpt_mixer_spec s{};
    int DK = 0, DV = 0;                 // padded head sizes (of one map)
    int maps = 1;
    const DBranch *v_first = nullptr;   // values are mixed with this branch's
    float v_share = 0.f, *sink = nullptr;
    float lambda = 0.f;                 // differential attention: from the four vectors below
    std::vector<float> lambda_part[4];
    float *q_norm = nullptr, *k_norm = nullptr;
    int q = -1, k = -1, v = -1, g = -1, a1 = -1, b = -1, g1 = -1;  // column offsets inside proj
    int za = -1, zg = -1;               // column offsets inside z
    int ra = 0, rg = 0;                 // padded ranks
    int out = 0;                        // column offset inside mixed
    int kv_layer = -1;
    uint64_t state_off = 0, conv_off = 0;
    void *w_a2 = nullptr, *w_g2 = nullptr;  // [heads * DK, ra], [heads * DV, rg]
    float *bias = nullptr, *a_log = nullptr, *norm = nullptr, *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr;
    uint64_t have = 0;
    float *bonus = nullptr, *lower = nullptr, *mu = nullptr;  // WKV [heads * DK], HGRN2 [heads * DK], WKV [5][width]
    int f = -1;                                               // HGRN2: forget gate's columns in proj
    // latent attention
    int dq = -1, dkv = -1, dkr = -1;      // columns in proj: query latent, key latent, rotated key part
    int DP = 0, DQ = 0, KR = 0, RR = 0, LDR = 0, qrp = 0;  // padded: head (unrotated), query head, latent, rotated part, page row, query latent
    int rot = -1;                         // which rotation of the model
    bool expand = false;                  // its head sizes have a written-out form
    void *w_uq = nullptr, *w_absorb = nullptr, *w_ukv = nullptr;  // [heads * DQ, qrp], [heads * KR, DP], [heads * (DP + DV), KR]
    float *dq_norm = nullptr, *dkv_norm = nullptr;
    float *removal_bias = nullptr;        // general delta [heads * DK]
    bool recurrent() const { return s.kind == JGPT_MIX_GLA || s.kind == JGPT_MIX_DELTA || s.kind == JGPT_MIX_HGRN2 || s.kind == JGPT_MIX_WKV || s.kind == JGPT_MIX_GENERAL_DELTA; }
    int cols() const { return s.heads * DV; }
};

struct DLayer {
    std::vector<DBranch> br;
    int ff = 0, ffp = 0, n_in = 0, n_out = 0, n_z = 0;
    int n_mix = 0, n_up = 0;                 // columns of the mixers in proj, of the first feed-forward product; gates lie behind
    int tanh_from = 0, tanh_to = 0;          // columns of proj with an activation
    float *post1 = nullptr, *post2 = nullptr, *share = nullptr, *bias_up = nullptr;
    uint64_t shift_off = 0, have_both = 0;
    bool v_source = false;                   // its projections stay for the layers that mix in its values
    void *w_in = nullptr, *w_out = nullptr, *w_gu = nullptr, *w_down = nullptr;
    float *n1w = nullptr, *n1b = nullptr, *n2w = nullptr, *n2b = nullptr;
    int ff_kind = 0;
    float act_p0 = 0.f, act_p1 = 0.f;
    float *ls1 = nullptr, *ls2 = nullptr, *dwa = nullptr;  // residual_mult x layer scale; depth average
    uint64_t have = 0;
    float *bias_in = nullptr;  // of the input projections
    // mixture of experts: [experts + identity (+ 1: the shared expert's gate), ldw], then all experts' up [effp, ldw] and down [ldw, effp]
    jgpt_moe_spec moe{};
    int effp = 0, sffp = 0, n_router = 0;
    void *w_router = nullptr, *w_eup = nullptr, *w_edown = nullptr, *w_sup = nullptr, *w_sdown = nullptr;
    float *correction = nullptr;
    uint64_t have_moe = 0;
    std::vector<uint8_t> have_expert;
    const DBranch *shift() const { return br[0].s.kind == JGPT_MIX_WKV ? &br[0] : nullptr; }  // its input projections read mixes
};

struct Decoder {
    Ctx *ctx = nullptr;
    jgpt_decoder_spec s{};
    bool f32 = false;
    int eb = 2, R = 0, ldw = 0;  // element bytes, rows per step, padded width
    std::vector<DLayer> L;
    void *embed = nullptr, *pos = nullptr, *head = nullptr;
    bool rms = false;
    const DBranch *v_first = nullptr;
    int v_first_ld = 0;
    std::vector<mix::Rotation> rots;
    std::vector<jgpt_mixer_spec> rot_specs;
    int max_window = 0;                // largest window of the latent layers (0: unbounded)
    int lat_min = 0, kvx_rows = 0;     // entries of at least lat_min tokens run latent attention written out, in kvx_rows workspace rows
    void *cq = nullptr, *q = nullptr, *qa = nullptr, *cx = nullptr, *kvx = nullptr;
    float *slots = nullptr;            // [layers + 1][rows][width] with depth averages
    float *enw = nullptr, *enb = nullptr, *fnw = nullptr, *fnb = nullptr;
    uint64_t have = 0;
    std::vector<KvLayerGeom> kv;
    uint64_t state_stride = 0;
    std::vector<void *> allocs;
    // workspace
    float *x = nullptr, *x_next = nullptr, *raw = nullptr, *chunk_ws = nullptr, *logits = nullptr;
    void *h = nullptr, *proj = nullptr, *proj_first = nullptr, *y = nullptr, *z = nullptr, *mixed = nullptr, *act = nullptr;
    // mixtures: activations of the experts' rows, their results, the same of the shared expert; routing
    void *e_act = nullptr, *e_out = nullptr, *s_act = nullptr, *s_out = nullptr;
    float *r_logits = nullptr;
    mix::RouteArgs route{};
    mix::PartNorm open{};              // what the layers left for the final norm
    float2 *row_inv = nullptr;         // 1 / root mean square of a row's queries and keys
    int *d_desc = nullptr, *h_desc = nullptr;
    int *d_next = nullptr, *h_next = nullptr;
    float *d_u = nullptr, *h_u = nullptr, *samp = nullptr;
    uint64_t chunk_ws_floats = 0;
    int long_min = 0;  // entries of at least this many tokens run their recurrences in chunks (0: none)
    int logit_rows = 0;
    // Decode steps (one token per entry, the picked ids as the only result) replayed as CUDA graphs from the second step of a
    // kind on.  The launches depend on the batch size, the length bucket and the pool's addresses: the key.
    struct Graph {
        const Pool *pool = nullptr;
        uint64_t generation = 0, last_use = 0;
        int n = 0, bucket = 0;
        cudaGraphExec_t exec = nullptr;
        bool failed = false;
    };
    std::vector<Graph> graphs;
    uint64_t graph_clock = 0;
    int use_graphs = 1, overlap = 1;  // JGPT_B200_DECODE_GRAPH, JGPT_B200_STEP_OVERLAP (0: off)
    float *capture = nullptr;  // host, [layers][rows][width] of the next step
    uint64_t capture_floats = 0;
};

Registry<Decoder> &decoder_registry() {
    static Registry<Decoder> r;
    return r;
}
int decoder_max_rows(const Decoder *d) { return d->R; }
int decoder_max_positions(const Decoder *d) { return d->s.max_positions; }
const int *decoder_next_tokens_device(const Decoder *d) { return d->d_next; }
Ctx *decoder_ctx(const Decoder *d) { return d->ctx; }

static int32_t dalloc(Decoder *d, void **p, uint64_t bytes) {
    JGPT_CUDA_TRY(cudaMalloc(p, std::max<uint64_t>(bytes, 16)));
    d->allocs.push_back(*p);
    JGPT_CUDA_TRY(cudaMemsetAsync(*p, 0, std::max<uint64_t>(bytes, 16), d->ctx->stream));
    return JGPT_OK;
}
#define TRY(expr)                        \
    do {                                 \
        const int32_t rc_ = (expr);      \
        if (rc_) return rc_;             \
    } while (0)

static void release(Decoder *d) {
    for (Decoder::Graph &g : d->graphs)
        if (g.exec) cudaGraphExecDestroy(g.exec);
    for (void *p : d->allocs) cudaFree(p);
    cudaFreeHost(d->h_desc), cudaFreeHost(d->h_next), cudaFreeHost(d->h_u);
    delete d;
}
int32_t decoder_destroy(Decoder *d) {
    JGPT_CUDA_TRY(make_current(d->ctx));
    cudaStreamSynchronize(d->ctx->stream);
    decoder_registry().remove(d);
    release(d);
    return JGPT_OK;
}

static mix::RecArgs rec_args(const DBranch &b) {
    mix::RecArgs a{};
    a.kind = b.s.kind == JGPT_MIX_DELTA ? mix::REC_DELTA : b.s.kind == JGPT_MIX_HGRN2 ? mix::REC_HGRN2 : b.s.kind == JGPT_MIX_WKV ? mix::REC_WKV
             : b.s.kind == JGPT_MIX_GENERAL_DELTA ? mix::REC_GENERAL : mix::REC_GLA;
    a.q_off = b.q, a.k_off = b.k, a.v_off = b.v, a.b_off = b.b, a.g_off = b.g, a.z_off = b.za, a.zg_off = b.zg;
    a.heads = b.s.heads, a.kv_heads = b.s.kv_heads, a.DK = b.DK, a.DV = b.DV, a.dim = b.s.dim, a.vdim = b.s.vdim;
    a.tau = b.s.tau, a.out_scale = b.s.out_scale, a.taps = b.s.kind == JGPT_MIX_DELTA ? b.s.taps : 0;
    a.conv_q = b.conv_q, a.conv_k = b.conv_k, a.conv_v = b.conv_v, a.decay_bias = b.bias, a.a_log = b.a_log, a.norm_w = b.norm;
    a.conv_off = b.conv_off, a.out_off = b.out;
    a.norm_stride = b.s.kind == JGPT_MIX_WKV || b.s.kind == JGPT_MIX_GENERAL_DELTA ? b.DV : 0, a.removal_bias = b.removal_bias, a.rate = b.s.decay_rate, a.bonus = b.bonus, a.lower = b.lower;
    if (b.s.kind == JGPT_MIX_HGRN2) a.z_off = b.f;
    return a;
}

// Source row i lands in row (i / rgroup) * rpad + i % rgroup, columns likewise: padding per head.
struct Grouping {
    int group = 0, pad = 0;  // group == 0: no grouping
    int at(int i) const { return group ? i / group * pad + i % group : i; }
};

static int32_t put_matrix(Decoder *d, void *dst, int ld, int row0, int col0, const float *src, int rows, int cols, Grouping rg, Grouping cg) {
    const int last = rg.at(rows - 1) + 1;
    const int width = cg.at(cols - 1) + 1;
    std::vector<uint8_t> buf((size_t)last * width * d->eb, 0);
    for (int r = 0; r < rows; r++)
        for (int c = 0; c < cols; c++) {
            const size_t o = (size_t)rg.at(r) * width + cg.at(c);
            const float v = src[(size_t)r * cols + c];
            if (d->f32) reinterpret_cast<float *>(buf.data())[o] = v;
            else reinterpret_cast<__nv_bfloat16 *>(buf.data())[o] = __float2bfloat16(v);
        }
    JGPT_CUDA_TRY(cudaMemcpy2DAsync(reinterpret_cast<uint8_t *>(dst) + ((size_t)row0 * ld + col0) * d->eb, (size_t)ld * d->eb, buf.data(),
                                    (size_t)width * d->eb, (size_t)width * d->eb, (size_t)last, cudaMemcpyHostToDevice, d->ctx->stream));
    JGPT_CUDA_TRY(cudaStreamSynchronize(d->ctx->stream));
    return JGPT_OK;
}
static int32_t put_floats(Decoder *d, float *dst, const float *src, int rows, int cols, Grouping rg) {
    std::vector<float> buf((size_t)(rg.at(rows - 1) + 1) * cols, 0.f);
    for (int r = 0; r < rows; r++) std::copy(src + (size_t)r * cols, src + (size_t)(r + 1) * cols, buf.begin() + (size_t)rg.at(r) * cols);
    JGPT_CUDA_TRY(cudaMemcpyAsync(dst, buf.data(), sizeof(float) * buf.size(), cudaMemcpyHostToDevice, d->ctx->stream));
    JGPT_CUDA_TRY(cudaStreamSynchronize(d->ctx->stream));
    return JGPT_OK;
}

// Angles of a rotation: frequencies on the device, the magnitude of cos and sin.
static int32_t add_rotation(Decoder *d, const jgpt_mixer_spec &s) {
    const int half = s.rot_dims / 2;
    std::vector<double> f((size_t)half);
    auto dim_of = [&](double turns) { return s.rot_dims * std::log(s.rot_original / (2 * M_PI * turns)) / (2 * std::log(s.rot_base)); };
    const bool yarn = s.rot_factor > 0;
    const double lo = yarn ? std::max(std::floor(dim_of(s.rot_fast)), 0.0) : 0, hi = yarn ? std::min(std::ceil(dim_of(s.rot_slow)), s.rot_dims - 1.0) : 0;
    for (int i = 0; i < half; i++) {
        f[(size_t)i] = std::pow(s.rot_base, -2.0 * i / s.rot_dims);
        if (!yarn) continue;
        const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
        f[(size_t)i] = f[(size_t)i] / s.rot_factor * ramp + f[(size_t)i] * (1 - ramp);
    }
    mix::Rotation r{};
    void *dev = nullptr;
    TRY(dalloc(d, &dev, sizeof(double) * f.size()));
    JGPT_CUDA_TRY(cudaMemcpyAsync(dev, f.data(), sizeof(double) * f.size(), cudaMemcpyHostToDevice, d->ctx->stream));
    JGPT_CUDA_TRY(cudaStreamSynchronize(d->ctx->stream));
    r.freq = (const double *)dev, r.half = half, r.mag = yarn ? (float)(0.1 * std::log(s.rot_factor) + 1.0) : 1.f;
    d->rots.push_back(r), d->rot_specs.push_back(s);
    return JGPT_OK;
}

static bool same_rotation(const jgpt_mixer_spec &x, const jgpt_mixer_spec &s) {
    return x.rot_dims == s.rot_dims && x.rot_base == s.rot_base && x.rot_factor == s.rot_factor && x.rot_original == s.rot_original &&
           x.rot_fast == s.rot_fast && x.rot_slow == s.rot_slow;
}
static int32_t find_rotation(Decoder *d, const jgpt_mixer_spec &s, int *rot) {
    for (size_t k = 0; k < d->rot_specs.size(); k++)
        if (same_rotation(d->rot_specs[k], s)) {
            *rot = (int)k;
            return JGPT_OK;
        }
    JGPT_REQUIRE(d->rots.size() < mix::kMaxRotations, JGPT_ERR_UNSUPPORTED, "more than %d different rotations", mix::kMaxRotations);
    *rot = (int)d->rots.size();
    return add_rotation(d, s);
}

// Sizes, weights and choice of a mixture.
static int32_t plan_moe(Decoder *d, DLayer &y, const jgpt_moe_spec &m, int index) {
    const int out = m.experts + m.identity;
    JGPT_REQUIRE(m.experts > 0 && m.identity >= 0 && m.ff > 0 && m.shared_ff >= 0 && m.groups > 0 && out % m.groups == 0 && m.keep > 0 && m.keep <= m.groups &&
                     m.top > 0 && m.top <= out / m.groups * m.keep,
                 JGPT_ERR_INVALID_ARGUMENT, "layer %d: %d + %d experts of %d in %d groups, %d of %d kept, shared part of %d", index, m.experts, m.identity, m.ff,
                 m.groups, m.top, m.keep, m.shared_ff);
    auto known = [](int act) { return act == JGPT_ACT_RELU || act == JGPT_ACT_RELU2 || act == JGPT_ACT_GELU_TANH; };
    JGPT_REQUIRE(known(m.act) && known(m.shared_act), JGPT_ERR_UNSUPPORTED, "layer %d: activations %d / %d", index, m.act, m.shared_act);
    JGPT_REQUIRE(d->s.norm_after, JGPT_ERR_UNSUPPORTED, "layer %d: mixtures of experts go with norms behind the sums", index);
    const uint64_t eb = d->eb, ldw = d->ldw;
    y.moe = m, y.effp = up(m.ff, 16), y.sffp = up(m.shared_ff, 16), y.n_router = out + (m.shared_ff ? 1 : 0);
    y.have_expert.assign((size_t)m.experts, 0);
    TRY(dalloc(d, &y.w_router, y.n_router * ldw * eb));
    TRY(dalloc(d, (void **)&y.correction, sizeof(float) * (uint64_t)out));
    TRY(dalloc(d, &y.w_eup, (uint64_t)m.experts * y.effp * ldw * eb));
    TRY(dalloc(d, &y.w_edown, (uint64_t)m.experts * y.effp * ldw * eb));
    if (m.shared_ff) {
        TRY(dalloc(d, &y.w_sup, y.sffp * ldw * eb));
        TRY(dalloc(d, &y.w_sdown, y.sffp * ldw * eb));
    }
    return JGPT_OK;
}

// Sizes, column layouts and device memory of one layer.
static int32_t plan_layer(Decoder *d, DLayer &y, const jgpt_layer_spec &ls, int index) {
    JGPT_REQUIRE(ls.n_branches >= 1 && ls.n_branches <= JGPT_MAX_BRANCHES, JGPT_ERR_INVALID_ARGUMENT, "layer %d: %d mixer branches", index,
                 ls.n_branches);
    JGPT_REQUIRE(ls.ff >= 0, JGPT_ERR_INVALID_ARGUMENT, "layer %d: feed-forward size %d", index, ls.ff);
    const int eb = d->eb, W = d->s.width;
    int in = 0, out = 0, zc = 0;
    auto seg = [&](int n) {
        const int o = in;
        in += up(n, 8);
        return o;
    };
    for (int i = 0; i < ls.n_branches; i++) {
        DBranch b;
        b.s = ls.branch[i];
        const jgpt_mixer_spec &s = b.s;
        JGPT_REQUIRE(s.heads > 0 && s.kv_heads > 0 && s.heads % s.kv_heads == 0 && s.dim > 0 && s.vdim > 0, JGPT_ERR_INVALID_ARGUMENT,
                     "layer %d: heads %d / %d, head sizes %d / %d", index, s.heads, s.kv_heads, s.dim, s.vdim);
        b.out = out;
        if (s.kind == JGPT_MIX_ATTENTION) {
            b.maps = std::max(s.maps, 1);
            JGPT_REQUIRE(b.maps <= 2 && s.gate >= 0 && s.gate <= 2, JGPT_ERR_UNSUPPORTED, "layer %d: %d attention maps, gate %d", index, b.maps, s.gate);
            JGPT_REQUIRE(mix::attn_padded_head(s.dim, s.vdim, b.maps, &b.DK, &b.DV), JGPT_ERR_UNSUPPORTED, "layer %d: head sizes %d / %d", index, s.dim, s.vdim);
            JGPT_REQUIRE(s.rot_dims >= 0 && s.rot_dims % 2 == 0 && s.rot_dims <= s.dim && (s.rot_dims == 0 || (s.rot_base > 1.0 && d->rms)), JGPT_ERR_INVALID_ARGUMENT,
                         "layer %d: rotation of %d of %d", index, s.rot_dims, s.dim);
            b.q = seg(s.heads * b.maps * b.DK), b.k = seg(s.kv_heads * b.maps * b.DK), b.v = seg(s.kv_heads * b.DV);
            if (s.gate) b.g = seg(s.gate == mix::GATE_HEAD ? s.heads : s.heads * b.DV);
            if (s.rot_dims) TRY(find_rotation(d, s, &b.rot));
            JGPT_REQUIRE(s.qk_norm >= 0 && s.qk_norm <= JGPT_QK_NORM_UNIT && (s.qk_norm != JGPT_QK_NORM_ALL || b.maps == 1), JGPT_ERR_UNSUPPORTED,
                         "layer %d: norm %d of queries and keys, %d maps", index, s.qk_norm, b.maps);
            JGPT_REQUIRE(s.window >= 0 && s.keep >= 0 && !(s.window && (s.chunk || b.maps > 1)) && (s.window || !s.keep) && s.sink >= 0 && s.sink <= JGPT_SINK_ZERO &&
                             (!s.sink || b.maps == 1),
                         JGPT_ERR_INVALID_ARGUMENT, "layer %d: window %d with %d kept, chunk %d, sink %d, %d maps", index, s.window, s.keep, s.chunk, s.sink, b.maps);
            if (s.qk_norm) {
                const bool all = s.qk_norm == JGPT_QK_NORM_ALL;
                TRY(dalloc(d, (void **)&b.q_norm, sizeof(float) * (uint64_t)(all ? s.heads * b.DK : s.dim)));
                TRY(dalloc(d, (void **)&b.k_norm, sizeof(float) * (uint64_t)(all ? s.kv_heads * b.DK : s.dim)));
                if (s.qk_norm == JGPT_QK_NORM_UNIT) {
                    const std::vector<float> ones((size_t)s.dim, 1.f);
                    for (float *p : {b.q_norm, b.k_norm}) TRY(put_floats(d, p, ones.data(), 1, s.dim, Grouping()));
                }
            }
            if (s.sink) TRY(dalloc(d, (void **)&b.sink, sizeof(float) * (uint64_t)s.heads));  // zeros
            if (s.v_mix) {
                JGPT_REQUIRE(ls.n_branches == 1, JGPT_ERR_UNSUPPORTED, "layer %d: mixed values stand alone in their layer", index);
                if (d->v_first) {
                    JGPT_REQUIRE(d->v_first->s.kv_heads * d->v_first->s.vdim == s.kv_heads * s.vdim, JGPT_ERR_INVALID_ARGUMENT,
                                 "layer %d: values of %d x %d are mixed with %d x %d", index, s.kv_heads, s.vdim, d->v_first->s.kv_heads, d->v_first->s.vdim);
                    b.v_first = d->v_first;
                } else {
                    y.v_source = true;
                }
            }
            b.kv_layer = (int)d->kv.size();
            KvLayerGeom geom;
            geom.heads = s.kv_heads, geom.dim = mix::page_row(b.maps * b.DK) + mix::page_row(b.DV), geom.parts = 1;
            d->kv.push_back(geom);
        } else if (s.kind == JGPT_MIX_GLA || s.kind == JGPT_MIX_DELTA) {
            const bool delta = s.kind == JGPT_MIX_DELTA;
            JGPT_REQUIRE(delta || s.kv_heads == s.heads, JGPT_ERR_UNSUPPORTED, "layer %d: gated linear attention has one key head per head", index);
            JGPT_REQUIRE(s.rank_a > 0 && (!delta || (s.rank_g > 0 && s.taps >= 1 && s.taps <= 8)) && (delta || s.tau > 0.f), JGPT_ERR_INVALID_ARGUMENT,
                         "layer %d: ranks %d / %d, %d convolution taps, tau %g", index, s.rank_a, s.rank_g, s.taps, (double)s.tau);
            b.DK = mix::rec_padded_key(s.dim), b.DV = mix::rec_padded_value(s.vdim);
            JGPT_REQUIRE(b.DK > 0 && b.DV > 0, JGPT_ERR_UNSUPPORTED, "layer %d: head sizes %d / %d", index, s.dim, s.vdim);
            b.q = seg(s.kv_heads * b.DK), b.k = seg(s.kv_heads * b.DK), b.v = seg(s.heads * b.DV);
            b.ra = up(s.rank_a, 8), b.a1 = seg(s.rank_a);
            b.za = zc, zc += s.heads * b.DK;
            TRY(dalloc(d, &b.w_a2, (uint64_t)s.heads * b.DK * b.ra * eb));
            TRY(dalloc(d, (void **)&b.bias, sizeof(float) * (uint64_t)s.heads * b.DK));
            TRY(dalloc(d, (void **)&b.norm, sizeof(float) * (uint64_t)b.DV));
            if (delta) {
                b.b = seg(s.heads);
                b.rg = up(s.rank_g, 8), b.g1 = seg(s.rank_g);
                b.zg = zc, zc += s.heads * b.DV;
                TRY(dalloc(d, &b.w_g2, (uint64_t)s.heads * b.DV * b.rg * eb));
                TRY(dalloc(d, (void **)&b.a_log, sizeof(float) * (uint64_t)s.heads));
                TRY(dalloc(d, (void **)&b.conv_q, sizeof(float) * (uint64_t)s.kv_heads * b.DK * s.taps));
                TRY(dalloc(d, (void **)&b.conv_k, sizeof(float) * (uint64_t)s.kv_heads * b.DK * s.taps));
                TRY(dalloc(d, (void **)&b.conv_v, sizeof(float) * (uint64_t)s.heads * b.DV * s.taps));
            } else {
                b.g = seg(s.heads * b.DV);
            }
            b.state_off = d->state_stride;
            d->state_stride += mix::rec_state_bytes(rec_args(b), eb, &b.conv_off);
        } else if (s.kind == JGPT_MIX_HGRN2 || s.kind == JGPT_MIX_WKV) {
            const bool wkv = s.kind == JGPT_MIX_WKV;
            JGPT_REQUIRE(s.kv_heads == s.heads && (!wkv || (s.vdim == s.dim && s.rank_a > 0)), JGPT_ERR_INVALID_ARGUMENT,
                         "layer %d: heads %d / %d, head sizes %d / %d, rank %d", index, s.heads, s.kv_heads, s.dim, s.vdim, s.rank_a);
            JGPT_REQUIRE(!wkv || (ls.n_branches == 1 && d->rms), JGPT_ERR_UNSUPPORTED, "layer %d: WKV stands alone in its layer, behind an RMS norm", index);
            b.DK = mix::rec_padded_key(s.dim), b.DV = wkv ? b.DK : mix::rec_padded_value(s.vdim);
            JGPT_REQUIRE(b.DK > 0 && b.DV > 0, JGPT_ERR_UNSUPPORTED, "layer %d: head sizes %d / %d", index, s.dim, s.vdim);
            const int hk = s.heads * b.DK;
            b.q = seg(hk);
            if (wkv) b.k = seg(hk);
            b.v = seg(s.heads * b.DV);
            TRY(dalloc(d, (void **)&b.bias, sizeof(float) * (uint64_t)hk));
            TRY(dalloc(d, (void **)&b.norm, sizeof(float) * (uint64_t)b.DV * (wkv ? s.heads : 1)));
            if (wkv) {
                b.g = seg(hk);
                b.ra = up(s.rank_a, 8), b.a1 = seg(s.rank_a);
                b.za = zc, zc += hk;
                TRY(dalloc(d, &b.w_a2, (uint64_t)hk * b.ra * eb));
                TRY(dalloc(d, (void **)&b.bonus, sizeof(float) * (uint64_t)hk));
                TRY(dalloc(d, (void **)&b.mu, sizeof(float) * 5 * (uint64_t)W));
            } else {
                b.f = seg(hk);
                TRY(dalloc(d, (void **)&b.lower, sizeof(float) * (uint64_t)hk));
            }
            b.state_off = d->state_stride;
            mix::RecArgs ra = rec_args(b);
            ra.shift_width = wkv ? W : 0;
            d->state_stride += mix::rec_state_bytes(ra, eb, &b.conv_off);
        } else if (s.kind == JGPT_MIX_GENERAL_DELTA) {
            JGPT_REQUIRE(s.kv_heads == s.heads && s.rank_a > 0 && s.decay_rate > 0.f && d->rms && ls.n_branches == 1, JGPT_ERR_INVALID_ARGUMENT,
                         "layer %d: heads %d / %d, rank %d, decay rate %g, %d branches", index, s.heads, s.kv_heads, s.rank_a, (double)s.decay_rate, ls.n_branches);
            b.DK = mix::rec_padded_key(s.dim), b.DV = mix::rec_padded_value(s.vdim);
            JGPT_REQUIRE(b.DK > 0 && b.DV > 0, JGPT_ERR_UNSUPPORTED, "layer %d: head sizes %d / %d", index, s.dim, s.vdim);
            const int hk = s.heads * b.DK, hv = s.heads * b.DV;
            b.q = seg(hk), b.k = seg(hk), b.v = seg(hv), b.g = seg(hv), b.b = seg(hk);
            b.ra = up(s.rank_a, 8), b.a1 = seg(s.rank_a), y.tanh_from = b.a1, y.tanh_to = b.a1 + b.ra;
            b.za = zc, zc += hk;
            TRY(dalloc(d, &b.w_a2, (uint64_t)hk * b.ra * eb));
            TRY(dalloc(d, (void **)&b.bias, sizeof(float) * (uint64_t)hk));
            TRY(dalloc(d, (void **)&b.removal_bias, sizeof(float) * (uint64_t)hk));
            TRY(dalloc(d, (void **)&b.norm, sizeof(float) * (uint64_t)hv));
            b.state_off = d->state_stride;
            d->state_stride += mix::rec_state_bytes(rec_args(b), eb, &b.conv_off);
        } else if (s.kind == JGPT_MIX_LATENT) {
            JGPT_REQUIRE(s.q_rank > 0 && s.kv_rank > 0 && s.window >= 0 && s.rot_dims > 0 && s.rot_dims % 2 == 0 && s.rot_dims <= s.rot_dim && s.rot_base > 1.0,
                         JGPT_ERR_INVALID_ARGUMENT, "layer %d: latents of %d / %d, window %d, rotation of %d / %d", index, s.q_rank, s.kv_rank, s.window,
                         s.rot_dims, s.rot_dim);
            b.KR = mix::latent_padded_rank(s.kv_rank), b.RR = mix::latent_padded_rot(s.rot_dim), b.LDR = b.KR + b.RR + 8;
            JGPT_REQUIRE(b.KR > 0 && b.RR > 0, JGPT_ERR_UNSUPPORTED, "layer %d: latent of %d, rotated part of %d", index, s.kv_rank, s.rot_dim);
            b.DP = up(s.dim, 8), b.DQ = b.DP + up(s.rot_dim, 8), b.DV = up(s.vdim, 8), b.qrp = up(s.q_rank, 8);
            b.expand = !d->f32 && mix::latent_expandable(s.dim, s.rot_dim, s.vdim);
            b.dq = seg(s.q_rank);
            if (s.kv_from == 0) {
                b.dkv = seg(s.kv_rank), b.dkr = seg(s.rot_dim);
                b.kv_layer = (int)d->kv.size();
                KvLayerGeom geom;
                geom.heads = 1, geom.dim = b.LDR, geom.parts = 1;
                d->kv.push_back(geom);
                TRY(dalloc(d, (void **)&b.dkv_norm, sizeof(float) * (uint64_t)s.kv_rank));
            } else {
                JGPT_REQUIRE(s.kv_from >= 1 && s.kv_from <= index, JGPT_ERR_INVALID_ARGUMENT, "layer %d reads the cache of layer %d", index, s.kv_from - 1);
                const DBranch *from = nullptr;
                for (const DBranch &x : d->L[(size_t)s.kv_from - 1].br)
                    if (x.s.kind == JGPT_MIX_LATENT && x.s.kv_from == 0) from = &x;
                JGPT_REQUIRE(from && from->s.kv_rank == s.kv_rank && from->s.rot_dim == s.rot_dim && same_rotation(from->s, s), JGPT_ERR_INVALID_ARGUMENT,
                             "layer %d: layer %d has no cache of its sizes and rotation", index, s.kv_from - 1);
                b.kv_layer = from->kv_layer;
            }
            TRY(find_rotation(d, s, &b.rot));
            TRY(dalloc(d, &b.w_uq, (uint64_t)s.heads * b.DQ * b.qrp * eb));
            TRY(dalloc(d, &b.w_absorb, (uint64_t)s.heads * b.KR * b.DP * eb));
            TRY(dalloc(d, &b.w_ukv, (uint64_t)s.heads * (b.DP + b.DV) * b.KR * eb));
            TRY(dalloc(d, (void **)&b.dq_norm, sizeof(float) * (uint64_t)s.q_rank));
        } else {
            return fail(JGPT_ERR_UNSUPPORTED, "layer %d: mixer kind %d", index, s.kind);
        }
        out += b.cols();
        y.br.push_back(b);
    }
    const bool gated = d->s.residual_gate;
    y.n_mix = in;
    if (gated) in += d->ldw;
    y.n_in = in, y.n_out = up(out, 8), y.n_z = zc, y.ff = ls.ff, y.ffp = up(ls.ff, 16), y.ff_kind = ls.ff_kind;
    JGPT_REQUIRE(ls.ff_kind >= JGPT_FF_GATED_GELU && ls.ff_kind <= JGPT_FF_RELU2, JGPT_ERR_UNSUPPORTED, "layer %d: feed-forward kind %d", index, ls.ff_kind);
    JGPT_REQUIRE((!d->s.norm_after && !d->s.norm_both) || !y.shift(), JGPT_ERR_UNSUPPORTED, "layer %d: WKV mixes inputs normed in front of it alone", index);
    const bool one_up = y.ff_kind == JGPT_FF_XIELU || y.ff_kind == JGPT_FF_RELU2;
    JGPT_REQUIRE(!gated || !y.ff || one_up, JGPT_ERR_UNSUPPORTED, "layer %d: a gated result of feed-forward kind %d", index, y.ff_kind);
    y.n_up = y.ffp + (gated ? d->ldw : 0);
    bool biased = gated;
    for (const DBranch &b : y.br) biased = biased || (b.s.kind == JGPT_MIX_ATTENTION && b.s.qkv_bias);
    biased = biased || y.tanh_to;  // columns beside those with an activation
    if (biased) TRY(dalloc(d, (void **)&y.bias_in, sizeof(float) * (uint64_t)y.n_in));
    if (y.ff && y.ff_kind == JGPT_FF_MOE) TRY(plan_moe(d, y, ls.moe, index));
    if (d->s.norm_both) {
        for (float **p : {&y.post1, &y.post2, &y.share}) TRY(dalloc(d, (void **)p, sizeof(float) * (uint64_t)d->ldw));
        if (gated && y.ff) TRY(dalloc(d, (void **)&y.bias_up, sizeof(float) * (uint64_t)y.n_up));
        y.shift_off = d->state_stride;
        if (d->s.token_shift) d->state_stride += up((int)(2 * sizeof(float)) * d->ldw, 256);
    }
    if (d->rms && !d->s.norm_after && !d->s.norm_both) {
        TRY(dalloc(d, (void **)&y.ls1, sizeof(float) * (uint64_t)W));
        TRY(dalloc(d, (void **)&y.ls2, sizeof(float) * (uint64_t)W));
        const std::vector<float> mult((size_t)W, d->s.residual_mult);
        for (float *p : {y.ls1, y.ls2}) TRY(put_floats(d, p, mult.data(), 1, W, Grouping()));
    }
    if (d->s.depth_average) TRY(dalloc(d, (void **)&y.dwa, sizeof(float) * (uint64_t)(index + 2)));
    TRY(dalloc(d, &y.w_in, (uint64_t)y.n_in * d->ldw * eb));
    TRY(dalloc(d, &y.w_out, (uint64_t)d->ldw * y.n_out * eb));
    TRY(dalloc(d, (void **)&y.n1w, sizeof(float) * (uint64_t)d->ldw));
    TRY(dalloc(d, (void **)&y.n1b, sizeof(float) * (uint64_t)W));
    if (y.ff) {
        if (y.ff_kind != JGPT_FF_MOE) {
            TRY(dalloc(d, &y.w_gu, (uint64_t)(one_up ? y.n_up : 2 * y.ffp) * d->ldw * eb));
            TRY(dalloc(d, &y.w_down, (uint64_t)d->ldw * y.ffp * eb));
        }
        TRY(dalloc(d, (void **)&y.n2w, sizeof(float) * (uint64_t)d->ldw));
        TRY(dalloc(d, (void **)&y.n2b, sizeof(float) * (uint64_t)W));
    }
    return JGPT_OK;
}

static size_t desc_ints(const Decoder *d) { return 40 * (size_t)d->R + 128; }

static int32_t build(Decoder *d, const jgpt_layer_spec *layers) {
    const uint64_t R = d->R, W = d->s.width, eb = d->eb;
    d->L.resize((size_t)d->s.n_layers);
    d->long_min = mix::rec_chunk_min_tokens(d->f32);
    d->rms = d->s.norm == JGPT_NORM_RMS;
    d->lat_min = env_int("JGPT_B200_LATENT_EXPAND_MIN", 64);
    int n_in = 8, n_z = 8, n_out = 8, ffp = 16, raw = 0, mixes = d->s.norm_both ? 2 : 1, cq = 0, lq = 0, lqa = 0, cxw = 0, kvx = 0;
    int top = 0, experts = 0, outputs = 0, effp = 0, sffp = 0, tiles = 0;
    bool latent = false, unbounded = false, expand = true;
    for (int i = 0; i < d->s.n_layers; i++) {
        DLayer &y = d->L[(size_t)i];
        TRY(plan_layer(d, y, layers[i], i));
        n_in = std::max(n_in, y.n_in), n_z = std::max(n_z, y.n_z), n_out = std::max(n_out, y.n_out), ffp = std::max(ffp, y.n_up);
        if (y.v_source) {
            d->v_first = &y.br[0], d->v_first_ld = y.n_in;
            TRY(dalloc(d, &d->proj_first, R * y.n_in * eb));
        }
        top = std::max(top, y.moe.top), experts = std::max(experts, y.moe.experts), outputs = std::max(outputs, y.n_router);
        effp = std::max(effp, y.effp), sffp = std::max(sffp, y.sffp);
        if (y.effp) tiles = std::max(tiles, std::min(y.moe.experts, d->R * y.moe.top) + d->R * y.moe.top / 16);
        for (const DBranch &b : y.br) {
            if (b.s.kind == JGPT_MIX_WKV) mixes = 5;
            if (b.s.kind == JGPT_MIX_LATENT) {
                latent = true, unbounded = unbounded || b.s.window == 0, d->max_window = std::max(d->max_window, b.s.window);
                cq = std::max(cq, b.qrp), lq = std::max(lq, b.s.heads * b.DQ), lqa = std::max(lqa, b.s.heads * b.KR), cxw = std::max(cxw, b.KR + b.RR);
                kvx = std::max(kvx, b.s.heads * (b.DP + b.DV)), expand = expand && b.expand;
            }
            if (!b.recurrent()) continue;
            raw = std::max(raw, b.s.heads * b.DV);
            if (const int t = d->long_min)
                d->chunk_ws_floats = std::max(d->chunk_ws_floats, (uint64_t)(d->R / mix::kRecChunk + d->R / t + 1) * b.s.heads *
                                                                      mix::rec_chunk_record_floats(rec_args(b).kind, b.DK, b.DV));
        }
    }
    TRY(dalloc(d, &d->embed, (uint64_t)d->s.vocab * d->ldw * eb));
    if (d->s.pos_table) TRY(dalloc(d, &d->pos, (uint64_t)d->s.max_positions * d->ldw * eb));
    if (d->s.head) TRY(dalloc(d, &d->head, (uint64_t)d->s.vocab * d->ldw * eb));
    for (float **p : {&d->enw, &d->enb, &d->fnw, &d->fnb}) TRY(dalloc(d, (void **)p, sizeof(float) * d->ldw));
    TRY(dalloc(d, (void **)&d->x, sizeof(float) * R * d->ldw));
    if (d->s.norm_both) {
        TRY(dalloc(d, (void **)&d->x_next, sizeof(float) * R * d->ldw));
        TRY(dalloc(d, &d->y, R * d->ldw * eb));
    }
    if (d->s.depth_average) TRY(dalloc(d, (void **)&d->slots, sizeof(float) * (d->L.size() + 1) * R * W));
    for (mix::Rotation &r : d->rots) TRY(dalloc(d, (void **)&r.out, sizeof(float2) * R * r.half));
    if (top) {
        const uint64_t copies = R * (uint64_t)top;
        mix::RouteArgs &r = d->route;
        TRY(dalloc(d, &d->e_act, copies * effp * eb));
        TRY(dalloc(d, &d->e_out, copies * d->ldw * eb));
        TRY(dalloc(d, &d->s_act, R * sffp * eb));
        TRY(dalloc(d, &d->s_out, R * (sffp ? d->ldw : 0) * eb));
        r.ld = up(outputs, 4), r.cap = d->R;
        TRY(dalloc(d, (void **)&d->r_logits, sizeof(float) * R * r.ld));
        TRY(dalloc(d, (void **)&r.slots, sizeof(mix::RouteSlot) * copies));
        TRY(dalloc(d, (void **)&r.row_weights, sizeof(float2) * R));
        TRY(dalloc(d, (void **)&r.list, sizeof(int) * R * experts));
        TRY(dalloc(d, (void **)&r.counts, sizeof(int) * (uint64_t)experts));
        TRY(dalloc(d, (void **)&r.offsets, sizeof(int) * (uint64_t)experts));
        TRY(dalloc(d, (void **)&r.ticket, sizeof(int)));
        TRY(dalloc(d, (void **)&r.tiles, sizeof(nt::RowTile) * (uint64_t)tiles));
        TRY(dalloc(d, (void **)&r.n_tiles, sizeof(int)));
        r.logits = d->r_logits;
    }
    if (unbounded) d->max_window = 0;
    if (!latent || !expand) d->lat_min = 0;
    if (latent) {
        TRY(dalloc(d, &d->cq, R * cq * eb));
        TRY(dalloc(d, &d->q, R * lq * eb));
        TRY(dalloc(d, &d->qa, R * lqa * eb));
        if (d->lat_min > 0) {
            d->kvx_rows = 2 * d->R;
            TRY(dalloc(d, &d->cx, (uint64_t)d->kvx_rows * cxw * eb));
            TRY(dalloc(d, &d->kvx, (uint64_t)d->kvx_rows * kvx * eb));
        }
    }
    TRY(dalloc(d, (void **)&d->row_inv, sizeof(float2) * R));
    TRY(dalloc(d, (void **)&d->raw, sizeof(float) * R * raw));
    TRY(dalloc(d, (void **)&d->chunk_ws, sizeof(float) * d->chunk_ws_floats));
    TRY(dalloc(d, &d->h, R * mixes * d->ldw * eb));
    TRY(dalloc(d, &d->proj, R * n_in * eb));
    TRY(dalloc(d, &d->z, R * n_z * eb));
    TRY(dalloc(d, &d->mixed, R * n_out * eb));
    TRY(dalloc(d, &d->act, R * ffp * eb));
    // logits of up to this many rows at a time
    d->logit_rows = (int)std::max<uint64_t>(1, std::min<uint64_t>(R, (64ull << 20) / (uint64_t)d->s.vocab));
    TRY(dalloc(d, (void **)&d->logits, sizeof(float) * (uint64_t)d->logit_rows * d->s.vocab));
    TRY(dalloc(d, (void **)&d->d_next, sizeof(int) * R));
    TRY(dalloc(d, (void **)&d->d_u, sizeof(float) * R));
    TRY(dalloc(d, (void **)&d->d_desc, sizeof(int) * desc_ints(d)));
    JGPT_CUDA_TRY(cudaHostAlloc(&d->h_desc, sizeof(int) * desc_ints(d), cudaHostAllocDefault));
    JGPT_CUDA_TRY(cudaHostAlloc(&d->h_next, sizeof(int) * R, cudaHostAllocDefault));
    JGPT_CUDA_TRY(cudaHostAlloc(&d->h_u, sizeof(float) * R, cudaHostAllocDefault));
    JGPT_CUDA_TRY(cudaStreamSynchronize(d->ctx->stream));
    return JGPT_OK;
}

// ------------------------------------------------------------------------------------------------
// Weights
// ------------------------------------------------------------------------------------------------
static uint64_t bit(int role) { return 1ull << role; }

static uint64_t needed_roles(const DBranch &b) {
    const jgpt_mixer_spec &s = b.s;
    if (s.kind == JGPT_MIX_GENERAL_DELTA)
        return bit(JGPT_W_Q) | bit(JGPT_W_K) | bit(JGPT_W_V) | bit(JGPT_W_G) | bit(JGPT_W_O) | bit(JGPT_W_A1) | bit(JGPT_W_A2) | bit(JGPT_W_DECAY_BIAS) |
               bit(JGPT_W_B) | bit(JGPT_W_B_BIAS) | bit(JGPT_W_HEAD_NORM);
    if (s.kind == JGPT_MIX_LATENT)
        return bit(JGPT_W_DQ) | bit(JGPT_W_DQ_NORM) | bit(JGPT_W_UQ) | bit(JGPT_W_UK) | bit(JGPT_W_UV) | bit(JGPT_W_O) |
               (s.kv_from ? 0 : bit(JGPT_W_DKV) | bit(JGPT_W_DKV_NORM));
    if (s.kind == JGPT_MIX_HGRN2)
        return bit(JGPT_W_Q) | bit(JGPT_W_F) | bit(JGPT_W_V) | bit(JGPT_W_O) | bit(JGPT_W_DECAY_BIAS) | bit(JGPT_W_LOWER) | bit(JGPT_W_HEAD_NORM);
    if (s.kind == JGPT_MIX_WKV)
        return bit(JGPT_W_Q) | bit(JGPT_W_K) | bit(JGPT_W_V) | bit(JGPT_W_G) | bit(JGPT_W_O) | bit(JGPT_W_A1) | bit(JGPT_W_A2) | bit(JGPT_W_DECAY_BIAS) |
               bit(JGPT_W_BONUS) | bit(JGPT_W_HEAD_NORM) | bit(JGPT_W_MU_R) | bit(JGPT_W_MU_K) | bit(JGPT_W_MU_V) | bit(JGPT_W_MU_G) | bit(JGPT_W_MU_W);
    uint64_t n = bit(JGPT_W_Q) | bit(JGPT_W_K) | bit(JGPT_W_V) | bit(JGPT_W_O);
    if (s.kind == JGPT_MIX_ATTENTION)
        return n | (s.gate ? bit(JGPT_W_G) : 0) | (s.qkv_bias ? bit(JGPT_W_Q_BIAS) | bit(JGPT_W_K_BIAS) | bit(JGPT_W_V_BIAS) : 0) |
               (s.qk_norm == JGPT_QK_NORM_HEAD || s.qk_norm == JGPT_QK_NORM_ALL ? bit(JGPT_W_Q_NORM) | bit(JGPT_W_K_NORM) : 0) | (s.sink == JGPT_SINK_LEARNED ? bit(JGPT_W_SINK) : 0) |
               (b.v_first ? bit(JGPT_W_VMIX) : 0) |
               (s.maps > 1 ? bit(JGPT_W_LQ1) | bit(JGPT_W_LK1) | bit(JGPT_W_LQ2) | bit(JGPT_W_LK2) : 0);
    n |= bit(JGPT_W_A1) | bit(JGPT_W_A2) | bit(JGPT_W_DECAY_BIAS) | bit(JGPT_W_HEAD_NORM);
    if (s.kind == JGPT_MIX_GLA) return n | bit(JGPT_W_G);
    return n | bit(JGPT_W_B) | bit(JGPT_W_A_LOG) | bit(JGPT_W_G1) | bit(JGPT_W_G2) | bit(JGPT_W_CONV_Q) | bit(JGPT_W_CONV_K) | bit(JGPT_W_CONV_V);
}

static int32_t missing_weights(const Decoder *d) {
    const uint64_t beta = d->rms ? 0 : ~0ull;
    const uint64_t top = bit(JGPT_W_EMBED) | (d->s.pos_table ? bit(JGPT_W_POS) : 0) | (d->s.head ? bit(JGPT_W_HEAD) : 0) | bit(JGPT_W_FINAL_NORM) |
                         (beta & bit(JGPT_W_FINAL_NORM_B)) | (d->s.embed_norm ? bit(JGPT_W_EMBED_NORM) | bit(JGPT_W_EMBED_NORM_B) : 0);
    JGPT_REQUIRE((d->have & top) == top, JGPT_ERR_ILLEGAL_STATE, "embedding or final norm weights are not set");
    for (size_t i = 0; i < d->L.size(); i++) {
        const DLayer &y = d->L[i];
        uint64_t n = bit(JGPT_W_NORM1) | (beta & bit(JGPT_W_NORM1_B)) | (d->s.layer_scale ? bit(JGPT_W_LS1) : 0) | (d->s.depth_average ? bit(JGPT_W_DWA) : 0);
        if (y.effp) {
            n |= bit(JGPT_W_NORM2);
            const uint64_t e = bit(JGPT_W_EXPERT_UP - 64) | bit(JGPT_W_EXPERT_DOWN - 64);
            const uint64_t m = bit(JGPT_W_ROUTER - 64) | bit(JGPT_W_CORRECTION - 64) |
                               (y.sffp ? bit(JGPT_W_SHARED_GATE - 64) | bit(JGPT_W_SHARED_UP - 64) | bit(JGPT_W_SHARED_DOWN - 64) : 0);
            JGPT_REQUIRE((y.have_moe & m) == m, JGPT_ERR_ILLEGAL_STATE, "router or shared expert of layer %zu are not set", i);
            for (size_t k = 0; k < y.have_expert.size(); k++)
                JGPT_REQUIRE((y.have_expert[k] & e) == e, JGPT_ERR_ILLEGAL_STATE, "expert %zu of layer %zu is not set", k, i);
        } else if (y.ff)
            n |= bit(JGPT_W_NORM2) | (beta & bit(JGPT_W_NORM2_B)) | bit(JGPT_W_FF_UP) | bit(JGPT_W_FF_DOWN) | (d->s.layer_scale ? bit(JGPT_W_LS2) : 0) |
                 (y.ff_kind == JGPT_FF_XIELU ? bit(JGPT_W_FF_ACT) : y.ff_kind == JGPT_FF_RELU2 ? 0 : bit(JGPT_W_FF_GATE));
        JGPT_REQUIRE((y.have & n) == n, JGPT_ERR_ILLEGAL_STATE, "norm or feed-forward weights of layer %zu are not set", i);
        if (d->s.norm_both) {
            auto at = [](int role) { return bit(role - JGPT_W_POST1); };
            const uint64_t m = at(JGPT_W_POST1) | (d->s.token_shift ? at(JGPT_W_SHIFT) : 0) | (d->s.residual_gate ? at(JGPT_W_RG1) | at(JGPT_W_RG1_B) : 0) |
                               (y.ff ? at(JGPT_W_POST2) | (d->s.residual_gate ? at(JGPT_W_RG2) | at(JGPT_W_RG2_B) : 0) : 0);
            JGPT_REQUIRE((y.have_both & m) == m, JGPT_ERR_ILLEGAL_STATE, "norms behind the parts, shift or gates of layer %zu are not set", i);
        }
        for (const DBranch &b : y.br)
            JGPT_REQUIRE((b.have & needed_roles(b)) == needed_roles(b), JGPT_ERR_ILLEGAL_STATE, "mixer weights of layer %zu are not set", i);
    }
    return JGPT_OK;
}

static int32_t set_tensor(Decoder *d, int layer, int branch, int role, const float *src, int rows, int cols) {
    const int W = d->s.width;
    auto shape = [&](int r, int c) -> int32_t {
        JGPT_REQUIRE(rows == r && cols == c, JGPT_ERR_INVALID_ARGUMENT, "layer %d branch %d tensor %d: [%d, %d] expected, got [%d, %d]", layer, branch,
                     role, r, c, rows, cols);
        return JGPT_OK;
    };
    const Grouping none;
    if (layer < 0) {
        switch (role) {
            case JGPT_W_EMBED: TRY(shape(d->s.vocab, W)); TRY(put_matrix(d, d->embed, d->ldw, 0, 0, src, rows, cols, none, none)); break;
            case JGPT_W_HEAD:
                JGPT_REQUIRE(d->head, JGPT_ERR_INVALID_ARGUMENT, "the logits come from the embedding");
                TRY(shape(d->s.vocab, W));
                TRY(put_matrix(d, d->head, d->ldw, 0, 0, src, rows, cols, none, none));
                break;
            case JGPT_W_POS: JGPT_REQUIRE(d->pos, JGPT_ERR_INVALID_ARGUMENT, "the model has no table of positions"); TRY(shape(d->s.max_positions, W)); TRY(put_matrix(d, d->pos, d->ldw, 0, 0, src, rows, cols, none, none)); break;
            case JGPT_W_EMBED_NORM: TRY(shape(1, W)); TRY(put_floats(d, d->enw, src, 1, W, none)); break;
            case JGPT_W_EMBED_NORM_B: TRY(shape(1, W)); TRY(put_floats(d, d->enb, src, 1, W, none)); break;
            case JGPT_W_FINAL_NORM: TRY(shape(1, W)); TRY(put_floats(d, d->fnw, src, 1, W, none)); break;
            case JGPT_W_FINAL_NORM_B: TRY(shape(1, W)); TRY(put_floats(d, d->fnb, src, 1, W, none)); break;
            default: return fail(JGPT_ERR_INVALID_ARGUMENT, "tensor %d does not belong to the model", role);
        }
        d->have |= bit(role);
        return JGPT_OK;
    }
    DLayer &y = d->L[(size_t)layer];
    if (branch >= JGPT_MAX_BRANCHES) {
        const int e = branch - JGPT_MAX_BRANCHES, ldw = d->ldw;
        JGPT_REQUIRE(e < (int)y.have_expert.size(), JGPT_ERR_OUT_OF_RANGE, "layer %d has %zu experts", layer, y.have_expert.size());
        auto expert = [&](void *base) { return reinterpret_cast<uint8_t *>(base) + (size_t)e * y.effp * ldw * d->eb; };
        if (role == JGPT_W_EXPERT_UP) {
            TRY(shape(y.moe.ff, W));
            TRY(put_matrix(d, expert(y.w_eup), ldw, 0, 0, src, rows, cols, none, none));
        } else if (role == JGPT_W_EXPERT_DOWN) {
            TRY(shape(W, y.moe.ff));
            TRY(put_matrix(d, expert(y.w_edown), y.effp, 0, 0, src, rows, cols, none, none));
        } else {
            return fail(JGPT_ERR_INVALID_ARGUMENT, "tensor %d does not belong to an expert", role);
        }
        y.have_expert[(size_t)e] |= (uint8_t)bit(role - 64);
        return JGPT_OK;
    }
    if (branch < 0 && role >= JGPT_W_POST1) {
        const bool ff_role = role == JGPT_W_POST2 || role == JGPT_W_RG2 || role == JGPT_W_RG2_B, gate = role >= JGPT_W_RG1;
        JGPT_REQUIRE(d->s.norm_both && role <= JGPT_W_RG2_B && (!ff_role || y.ff) && (!gate || d->s.residual_gate) && (role != JGPT_W_SHIFT || d->s.token_shift),
                     JGPT_ERR_INVALID_ARGUMENT, "tensor %d does not belong to layer %d", role, layer);
        switch (role) {
            case JGPT_W_POST1: TRY(shape(1, W)); TRY(put_floats(d, y.post1, src, 1, W, none)); break;
            case JGPT_W_POST2: TRY(shape(1, W)); TRY(put_floats(d, y.post2, src, 1, W, none)); break;
            case JGPT_W_SHIFT: TRY(shape(1, W)); TRY(put_floats(d, y.share, src, 1, W, none)); break;
            case JGPT_W_RG1: TRY(shape(W, W)); TRY(put_matrix(d, y.w_in, d->ldw, y.n_mix, 0, src, W, W, none, none)); break;
            case JGPT_W_RG1_B: TRY(shape(1, W)); TRY(put_floats(d, y.bias_in + y.n_mix, src, 1, W, none)); break;
            case JGPT_W_RG2: TRY(shape(W, W)); TRY(put_matrix(d, y.w_gu, d->ldw, y.ffp, 0, src, W, W, none, none)); break;
            case JGPT_W_RG2_B: TRY(shape(1, W)); TRY(put_floats(d, y.bias_up + y.ffp, src, 1, W, none)); break;
        }
        y.have_both |= bit(role - JGPT_W_POST1);
        return JGPT_OK;
    }
    if (branch < 0 && role >= 64) {
        const int out = y.moe.experts + y.moe.identity;
        const bool shared = role == JGPT_W_SHARED_GATE || role == JGPT_W_SHARED_UP || role == JGPT_W_SHARED_DOWN;
        JGPT_REQUIRE(y.effp && role < 128 && (!shared || y.sffp), JGPT_ERR_INVALID_ARGUMENT, "layer %d has no %s", layer, shared ? "shared expert" : "mixture of experts");
        switch (role) {
            case JGPT_W_ROUTER: TRY(shape(out, W)); TRY(put_matrix(d, y.w_router, d->ldw, 0, 0, src, rows, cols, none, none)); break;
            case JGPT_W_SHARED_GATE: TRY(shape(1, W)); TRY(put_matrix(d, y.w_router, d->ldw, out, 0, src, rows, cols, none, none)); break;
            case JGPT_W_CORRECTION: TRY(shape(1, out)); TRY(put_floats(d, y.correction, src, 1, out, none)); break;
            case JGPT_W_SHARED_UP: TRY(shape(y.moe.shared_ff, W)); TRY(put_matrix(d, y.w_sup, d->ldw, 0, 0, src, rows, cols, none, none)); break;
            case JGPT_W_SHARED_DOWN: TRY(shape(W, y.moe.shared_ff)); TRY(put_matrix(d, y.w_sdown, y.sffp, 0, 0, src, rows, cols, none, none)); break;
            default: return fail(JGPT_ERR_INVALID_ARGUMENT, "tensor %d does not belong to a layer", role);
        }
        y.have_moe |= bit(role - 64);
        return JGPT_OK;
    }
    if (branch < 0) {
        const Grouping pair{16, 32};
        const bool ff_role = role == JGPT_W_FF_ACT || role == JGPT_W_LS2 || role == JGPT_W_FF_GATE || role == JGPT_W_FF_UP || role == JGPT_W_FF_DOWN || role == JGPT_W_NORM2 || role == JGPT_W_NORM2_B;
        const bool ff_norm = role == JGPT_W_NORM2 || role == JGPT_W_NORM2_B;
        JGPT_REQUIRE(!ff_role || (y.ff && (ff_norm || !y.effp)), JGPT_ERR_INVALID_ARGUMENT, "layer %d has no such feed-forward part", layer);
        switch (role) {
            case JGPT_W_NORM1: TRY(shape(1, W)); TRY(put_floats(d, y.n1w, src, 1, W, none)); break;
            case JGPT_W_NORM1_B: TRY(shape(1, W)); TRY(put_floats(d, y.n1b, src, 1, W, none)); break;
            case JGPT_W_NORM2: TRY(shape(1, W)); TRY(put_floats(d, y.n2w, src, 1, W, none)); break;
            case JGPT_W_NORM2_B: TRY(shape(1, W)); TRY(put_floats(d, y.n2b, src, 1, W, none)); break;
            case JGPT_W_LS1:
            case JGPT_W_LS2: {
                JGPT_REQUIRE(d->s.layer_scale, JGPT_ERR_INVALID_ARGUMENT, "the model has no layer scales");
                TRY(shape(1, W));
                std::vector<float> v(src, src + W);
                for (float &x : v) x *= d->s.residual_mult;
                TRY(put_floats(d, role == JGPT_W_LS1 ? y.ls1 : y.ls2, v.data(), 1, W, none));
                break;
            }
            case JGPT_W_DWA:
                JGPT_REQUIRE(y.dwa, JGPT_ERR_INVALID_ARGUMENT, "the model has no depth averages");
                TRY(shape(1, layer + 2));
                TRY(put_floats(d, y.dwa, src, 1, cols, none));
                break;
            case JGPT_W_FF_ACT: {
                JGPT_REQUIRE(y.ff_kind == JGPT_FF_XIELU, JGPT_ERR_INVALID_ARGUMENT, "layer %d: the activation has no parameters", layer);
                TRY(shape(1, 2));
                auto softplus = [](double z) { return std::max(z, 0.0) + std::log1p(std::exp(-std::fabs(z))); };
                y.act_p0 = (float)softplus(src[0]), y.act_p1 = (float)(0.5 + softplus(src[1]));
                break;
            }
            case JGPT_W_FF_GATE:
            case JGPT_W_FF_UP: {
                if (y.ff_kind == JGPT_FF_XIELU || y.ff_kind == JGPT_FF_RELU2) {
                    JGPT_REQUIRE(role == JGPT_W_FF_UP, JGPT_ERR_INVALID_ARGUMENT, "layer %d: the feed-forward part has no gate", layer);
                    TRY(shape(y.ff, W));
                    TRY(put_matrix(d, y.w_gu, d->ldw, 0, 0, src, rows, cols, none, none));
                    break;
                }
                // rows in groups of 16: gate, linear, gate, ... (two strided copies would overwrite each other's gaps)
                TRY(shape(y.ff, W));
                for (int r = 0; r < rows; r += 16)
                    TRY(put_matrix(d, y.w_gu, d->ldw, pair.at(r) + (role == JGPT_W_FF_UP ? 16 : 0), 0, src + (size_t)r * W, std::min(16, rows - r), W,
                                   none, none));
                break;
            }
            case JGPT_W_FF_DOWN: TRY(shape(W, y.ff)); TRY(put_matrix(d, y.w_down, y.ffp, 0, 0, src, rows, cols, none, none)); break;
            default: return fail(JGPT_ERR_INVALID_ARGUMENT, "tensor %d does not belong to a layer", role);
        }
        y.have |= bit(role);
        return JGPT_OK;
    }
    JGPT_REQUIRE(branch < (int)y.br.size(), JGPT_ERR_OUT_OF_RANGE, "layer %d has %zu mixer branches", layer, y.br.size());
    DBranch &b = y.br[(size_t)branch];
    const jgpt_mixer_spec &s = b.s;
    JGPT_REQUIRE(role >= 0 && role < 64 && (needed_roles(b) & bit(role)), JGPT_ERR_INVALID_ARGUMENT, "tensor %d does not belong to mixer kind %d", role,
                 s.kind);
    const bool att = s.kind == JGPT_MIX_ATTENTION;
    const Grouping kg{s.dim, b.DK}, vg{s.vdim, b.DV};
    const int vheads = att ? s.kv_heads : s.heads, qheads = att ? s.heads * b.maps : s.kv_heads, kheads = s.kv_heads * (att ? b.maps : 1);
    auto into_proj = [&](int off, int n, Grouping g) -> int32_t {
        TRY(shape(n, W));
        return put_matrix(d, y.w_in, d->ldw, off, 0, src, rows, cols, g, none);
    };
    switch (role) {
        case JGPT_W_Q: TRY(into_proj(b.q, qheads * s.dim, kg)); break;
        case JGPT_W_K: TRY(into_proj(b.k, kheads * s.dim, kg)); break;
        case JGPT_W_V: TRY(into_proj(b.v, vheads * s.vdim, vg)); break;
        case JGPT_W_G:
            if (att && s.gate == mix::GATE_HEAD) TRY(into_proj(b.g, s.heads, none));
            else TRY(into_proj(b.g, s.heads * s.vdim, vg));
            break;
        case JGPT_W_Q_BIAS: TRY(shape(1, qheads * s.dim)); TRY(put_floats(d, y.bias_in + b.q, src, cols, 1, kg)); break;
        case JGPT_W_K_BIAS: TRY(shape(1, kheads * s.dim)); TRY(put_floats(d, y.bias_in + b.k, src, cols, 1, kg)); break;
        case JGPT_W_V_BIAS: TRY(shape(1, vheads * s.vdim)); TRY(put_floats(d, y.bias_in + b.v, src, cols, 1, vg)); break;
        case JGPT_W_Q_NORM:
        case JGPT_W_K_NORM: {
            float *dst = role == JGPT_W_Q_NORM ? b.q_norm : b.k_norm;
            const bool all = s.qk_norm == JGPT_QK_NORM_ALL;
            TRY(shape(1, all ? (role == JGPT_W_Q_NORM ? s.heads : s.kv_heads) * s.dim : s.dim));
            TRY(all ? put_floats(d, dst, src, cols, 1, kg) : put_floats(d, dst, src, 1, cols, none));
            break;
        }
        case JGPT_W_SINK: TRY(shape(1, s.heads)); TRY(put_floats(d, b.sink, src, 1, cols, none)); break;
        case JGPT_W_VMIX: TRY(shape(1, 1)); b.v_share = src[0]; break;
        case JGPT_W_B_BIAS: TRY(shape(1, s.heads * s.dim)); TRY(put_floats(d, b.removal_bias, src, cols, 1, kg)); break;
        case JGPT_W_LQ1:
        case JGPT_W_LK1:
        case JGPT_W_LQ2:
        case JGPT_W_LK2: {
            TRY(shape(1, s.dim));
            b.lambda_part[role - JGPT_W_LQ1].assign(src, src + s.dim);
            double dot[2] = {0, 0};
            for (int k = 0; k < 2; k++)
                if (const std::vector<float> &u = b.lambda_part[2 * k], &v = b.lambda_part[2 * k + 1]; u.size() == v.size())
                    for (size_t j = 0; j < u.size(); j++) dot[k] += (double)u[j] * v[j];
            b.lambda = (float)(std::exp(dot[0]) - std::exp(dot[1]) + (double)s.diff);
            break;
        }
        case JGPT_W_B:
            if (s.kind == JGPT_MIX_GENERAL_DELTA) TRY(into_proj(b.b, s.heads * s.dim, kg));
            else TRY(into_proj(b.b, s.heads, none));
            break;
        case JGPT_W_A1: TRY(into_proj(b.a1, s.rank_a, none)); break;
        case JGPT_W_G1: TRY(into_proj(b.g1, s.rank_g, none)); break;
        case JGPT_W_A2: TRY(shape(s.heads * s.dim, s.rank_a)); TRY(put_matrix(d, b.w_a2, b.ra, 0, 0, src, rows, cols, kg, none)); break;
        case JGPT_W_G2: TRY(shape(s.heads * s.vdim, s.rank_g)); TRY(put_matrix(d, b.w_g2, b.rg, 0, 0, src, rows, cols, vg, none)); break;
        case JGPT_W_DECAY_BIAS: TRY(shape(1, s.heads * s.dim)); TRY(put_floats(d, b.bias, src, cols, 1, kg)); break;
        case JGPT_W_A_LOG: TRY(shape(1, s.heads)); TRY(put_floats(d, b.a_log, src, 1, cols, none)); break;
        case JGPT_W_HEAD_NORM:
            if (s.kind == JGPT_MIX_WKV || s.kind == JGPT_MIX_GENERAL_DELTA) {
                TRY(shape(1, s.heads * s.vdim));
                TRY(put_floats(d, b.norm, src, cols, 1, vg));
            } else {
                TRY(shape(1, s.vdim));
                TRY(put_floats(d, b.norm, src, 1, cols, none));
            }
            break;
        case JGPT_W_BONUS: TRY(shape(s.heads, s.dim)); TRY(put_floats(d, b.bonus, src, rows * cols, 1, kg)); break;
        case JGPT_W_LOWER: TRY(shape(1, s.heads * s.dim)); TRY(put_floats(d, b.lower, src, cols, 1, kg)); break;
        case JGPT_W_F: TRY(into_proj(b.f, s.heads * s.dim, kg)); break;
        case JGPT_W_MU_R:
        case JGPT_W_MU_K:
        case JGPT_W_MU_V:
        case JGPT_W_MU_G:
        case JGPT_W_MU_W: TRY(shape(1, W)); TRY(put_floats(d, b.mu + (size_t)(role - JGPT_W_MU_R) * W, src, 1, W, none)); break;
        case JGPT_W_DQ: TRY(into_proj(b.dq, s.q_rank, none)); break;
        case JGPT_W_DQ_NORM: TRY(shape(1, s.q_rank)); TRY(put_floats(d, b.dq_norm, src, 1, cols, none)); break;
        case JGPT_W_DKV_NORM: TRY(shape(1, s.kv_rank)); TRY(put_floats(d, b.dkv_norm, src, 1, cols, none)); break;
        case JGPT_W_DKV:
            TRY(shape(s.kv_rank + s.rot_dim, W));
            TRY(put_matrix(d, y.w_in, d->ldw, b.dkv, 0, src, s.kv_rank, W, none, none));
            TRY(put_matrix(d, y.w_in, d->ldw, b.dkr, 0, src + (size_t)s.kv_rank * W, s.rot_dim, W, none, none));
            break;
        case JGPT_W_UQ:
            TRY(shape(s.heads * (s.dim + s.rot_dim), s.q_rank));
            for (int h = 0; h < s.heads; h++) {
                const float *hs = src + (size_t)h * (s.dim + s.rot_dim) * s.q_rank;
                TRY(put_matrix(d, b.w_uq, b.qrp, h * b.DQ, 0, hs, s.dim, s.q_rank, none, none));
                TRY(put_matrix(d, b.w_uq, b.qrp, h * b.DQ + b.DP, 0, hs + (size_t)s.dim * s.q_rank, s.rot_dim, s.q_rank, none, none));
            }
            break;
        case JGPT_W_UK: {
            TRY(shape(s.heads * s.dim, s.kv_rank));
            std::vector<float> t((size_t)s.kv_rank * s.dim);
            for (int h = 0; h < s.heads; h++) {
                for (int i = 0; i < s.dim; i++)
                    for (int c = 0; c < s.kv_rank; c++) t[(size_t)c * s.dim + i] = src[((size_t)h * s.dim + i) * s.kv_rank + c];
                TRY(put_matrix(d, b.w_absorb, b.DP, h * b.KR, 0, t.data(), s.kv_rank, s.dim, none, none));
                TRY(put_matrix(d, b.w_ukv, b.KR, h * b.DP, 0, src + (size_t)h * s.dim * s.kv_rank, s.dim, s.kv_rank, none, none));
            }
            break;
        }
        case JGPT_W_UV:
            TRY(shape(s.heads * s.vdim, s.kv_rank));
            for (int h = 0; h < s.heads; h++)
                TRY(put_matrix(d, b.w_ukv, b.KR, s.heads * b.DP + h * b.DV, 0, src + (size_t)h * s.vdim * s.kv_rank, s.vdim, s.kv_rank, none, none));
            break;
        case JGPT_W_CONV_Q: TRY(shape(s.kv_heads * s.dim, s.taps)); TRY(put_floats(d, b.conv_q, src, rows, cols, kg)); break;
        case JGPT_W_CONV_K: TRY(shape(s.kv_heads * s.dim, s.taps)); TRY(put_floats(d, b.conv_k, src, rows, cols, kg)); break;
        case JGPT_W_CONV_V: TRY(shape(s.heads * s.vdim, s.taps)); TRY(put_floats(d, b.conv_v, src, rows, cols, vg)); break;
        case JGPT_W_O: TRY(shape(W, s.heads * s.vdim)); TRY(put_matrix(d, y.w_out, y.n_out, 0, b.out, src, rows, cols, none, vg)); break;
        default: return fail(JGPT_ERR_INVALID_ARGUMENT, "tensor %d", role);
    }
    b.have |= bit(role);
    return JGPT_OK;
}

// ------------------------------------------------------------------------------------------------
// The step
// ------------------------------------------------------------------------------------------------
int32_t decoder_check_pool(const Decoder *d, const Pool *p) {
    JGPT_REQUIRE(p, JGPT_ERR_BAD_HANDLE, "bad kvpool handle");
    JGPT_REQUIRE(p->ctx == d->ctx, JGPT_ERR_INVALID_ARGUMENT, "model and KV pool live on different contexts");
    bool ok = p->layered && p->elem_bytes == d->eb && p->state_stride == d->state_stride && p->vlayers.size() == d->kv.size();
    for (size_t i = 0; ok && i < d->kv.size(); i++)
        ok = p->vlayers[i].heads == d->kv[i].heads && p->vlayers[i].dim == d->kv[i].dim && p->vlayers[i].parts == d->kv[i].parts;
    JGPT_REQUIRE(ok, JGPT_ERR_INVALID_ARGUMENT, "KV pool geometry does not match the model");
    return JGPT_OK;
}

// pdl (every launch of a step but the first): bit 0 = the kernel may start while its predecessor drains and waits itself
// before it touches anything a kernel of this step writes; bit 1 = it lets its successor do the same.
static int32_t product(Decoder *d, const nt::Problem *p, int n, nt::Epilogue epi, int pdl) {
    return d->f32 ? nt::launch_f32(p, n, epi, d->ctx->stream) : nt::launch_bf16(d->ctx, p, n, epi, pdl, d->ctx->stream);
}

// The residual in front of layer i (the number of layers: in front of the final norm).
static mix::RowSource residual(const Decoder *d, size_t i) {
    mix::RowSource r{};
    if (i == 0) {
        r.embed = d->embed, r.ld_embed = d->ldw, r.vocab = d->s.vocab, r.embed_scale = d->s.embed_scale;
        for (const mix::Rotation &x : d->rots) r.rot[r.n_rot++] = x;
    } else if (d->s.depth_average) {
        r.slots = d->slots, r.slot_stride = (uint64_t)d->R * d->s.width, r.weights = d->L[i - 1].dwa, r.n_slots = (int)i + 1;
    } else {
        r.slots = d->x, r.n_slots = 1;
    }
    return r;
}

// Groups of long entries whose keys fit the workspace together.
struct LatentBatch {
    int first, n, rows, max_keys, tile0, n_tiles;
};

static int32_t enqueue_latent(Decoder *d, Pool *p, const mix::StepDesc &sd, const std::vector<LatentBatch> &batches, const DLayer &y, const DBranch &b, int pdl) {
    const int R = sd.rows, eb = d->eb, H = b.s.heads;
    cudaStream_t st = d->ctx->stream;
    mix::LatentArgs a{};
    a.proj = d->proj, a.ldp = y.n_in, a.dq_off = b.dq, a.c_off = b.dkv, a.r_off = b.dkr;
    a.q_rank = b.s.q_rank, a.kv_rank = b.s.kv_rank, a.rot_dim = b.s.rot_dim, a.half = b.s.rot_dims / 2, a.eps = d->s.eps, a.scale = b.s.score_scale;
    a.dq_norm = b.dq_norm, a.dkv_norm = b.dkv_norm, a.cq = d->cq, a.ldcq = b.qrp, a.own_cache = b.s.kv_from == 0;
    a.KR = b.KR, a.RR = b.RR, a.LDR = b.LDR;
    a.kv = p->vkv + p->vlayers[(size_t)b.kv_layer].offset, a.table = p->d_table, a.n_blocks = p->n_blocks, a.mbs = p->max_blocks_per_seq;
    a.cs = d->rots[(size_t)b.rot].out, a.q = d->q, a.ldq = H * b.DQ, a.DQ = b.DQ, a.DP = b.DP, a.dim = b.s.dim, a.qa = d->qa;
    a.heads = H, a.window = b.s.window, a.cx = d->cx, a.kvx = d->kvx, a.ldx = H * (b.DP + b.DV), a.DVm = b.DV, a.vdim = b.s.vdim;
    a.out = d->mixed, a.ldo = y.n_out, a.out_off = b.out, a.sm_count = d->ctx->sm_count, a.status = d->ctx->d_status;
    auto at = [&](void *base, size_t elements) { return reinterpret_cast<uint8_t *>(base) + elements * eb; };
    TRY(mix::launch_latent_prep(d->f32, sd, a, pdl, st));
    nt::Problem q{d->cq, b.w_uq, d->q, nullptr, R, a.ldq, b.qrp, b.qrp, b.qrp, a.ldq, 1.f};
    TRY(product(d, &q, 1, nt::EPI_STORE, pdl));
    if (const int n = sd.lat_hi - sd.lat_lo; n > 0) {
        const size_t r0 = (size_t)sd.lat_lo;
        nt::Problem in{at(d->q, r0 * a.ldq), b.w_absorb, at(d->qa, r0 * H * b.KR), nullptr, n, H * b.KR, b.DP, a.ldq, b.DP, H * b.KR, 1.f};
        in.seg_n = b.KR, in.a_seg = b.DQ;
        TRY(product(d, &in, 1, nt::EPI_STORE, pdl));
        TRY(mix::launch_latent_attention(d->f32, sd, a, pdl, st));
        nt::Problem out{at(d->qa, r0 * H * b.KR), at(b.w_ukv, (size_t)H * b.DP * b.KR), at(d->mixed, r0 * y.n_out + b.out), nullptr, n, H * b.DV, b.KR,
                        H * b.KR, b.KR, y.n_out, 1.f};
        out.seg_n = b.DV, out.a_seg = b.KR;
        TRY(product(d, &out, 1, nt::EPI_STORE, pdl));
    }
    for (const LatentBatch &g : batches) {
        TRY(mix::launch_latent_gather(sd, a, g.first, g.n, g.max_keys, pdl, st));
        nt::Problem kv{d->cx, b.w_ukv, d->kvx, nullptr, g.rows, a.ldx, b.KR, b.KR + b.RR, b.KR, a.ldx, 1.f};
        TRY(product(d, &kv, 1, nt::EPI_STORE, pdl));
        TRY(mix::launch_latent_tiles(sd, a, g.tile0, g.n_tiles, pdl, st));
    }
    return JGPT_OK;
}

// Router, choice, products of the experts; the norm kernel adds what m says.
static int32_t enqueue_moe(Decoder *d, const DLayer &y, int R, int pdl, mix::MoeSum &m) {
    const int ldw = d->ldw, T = nt::group_tile_rows(d->f32, R, y.moe.top, y.moe.experts);
    auto act = [](int a) { return a == JGPT_ACT_RELU2 ? nt::ACT_RELU2 : (a == JGPT_ACT_RELU ? nt::ACT_RELU : nt::ACT_GELU); };
    mix::RouteArgs r = d->route;
    nt::Problem logits{d->h, y.w_router, d->r_logits, nullptr, R, y.n_router, ldw, ldw, ldw, r.ld, 1.f};
    TRY(product(d, &logits, 1, nt::EPI_SCALE_F32, pdl));
    r.experts = y.moe.experts, r.identity = y.moe.identity, r.top = y.moe.top, r.groups = y.moe.groups, r.keep = y.moe.keep, r.shared = y.sffp ? 1 : 0;
    r.correction = y.correction, r.tile_rows = T, r.max_tiles = std::min(y.moe.experts, R * y.moe.top) + R * y.moe.top / T;
    TRY(mix::launch_route(r, R, pdl, d->ctx->stream));
    nt::RowGroups g;
    g.tiles = r.tiles, g.n_tiles = r.n_tiles, g.max_tiles = r.max_tiles, g.rows = T, g.n_groups = y.moe.experts, g.a_rows = R, g.w_group = (long long)y.effp * ldw;
    const bool copied = T == nt::kLargeTile;  // the tcgen05 product reads its rows group by group, from the place of the results to come
    if (copied) TRY(mix::launch_moe_gather(r, d->h, d->e_out, ldw, pdl, d->ctx->stream));
    nt::Problem in[2] = {{d->h, y.w_eup, d->e_act, r.list, R, y.effp, ldw, ldw, ldw, y.effp, 1.f}, {d->h, y.w_sup, d->s_act, nullptr, R, y.sffp, ldw, ldw, ldw, y.sffp, 1.f}};
    if (copied) in[0].A = d->e_out, in[0].rowsel = nullptr, g.a_rows = R * y.moe.top;
    in[0].grp = g, in[0].act = act(y.moe.act), in[1].act = act(y.moe.shared_act);
    TRY(product(d, in, y.sffp ? 2 : 1, nt::EPI_ACT, pdl));
    g.a_rows = R * y.moe.top, g.early = true;
    nt::Problem out[2] = {{d->e_act, y.w_edown, d->e_out, nullptr, R, ldw, y.effp, y.effp, y.effp, ldw, 1.f},
                          {d->s_act, y.w_sdown, d->s_out, nullptr, R, ldw, y.sffp, y.sffp, y.sffp, ldw, 1.f}};
    out[0].grp = g;
    TRY(product(d, out, y.sffp ? 2 : 1, nt::EPI_STORE, pdl));
    m.out = d->e_out, m.shared = y.sffp ? d->s_out : nullptr, m.ld = ldw, m.top = y.moe.top, m.cap = r.cap, m.slots = r.slots, m.row_weights = r.row_weights;
    m.offsets = r.offsets, m.alpha = d->s.residual_scale;
    return JGPT_OK;
}

static void set_activation(const DLayer &y, nt::Problem &p) {
    switch (y.ff_kind) {
        case JGPT_FF_XIELU: p.act = nt::ACT_XIELU, p.p0 = y.act_p0, p.p1 = y.act_p1; break;
        case JGPT_FF_RELU2: p.act = nt::ACT_RELU2; break;
        case JGPT_FF_GATED_RELU: p.act = nt::ACT_RELU; break;
        default: p.act = nt::ACT_GELU;
    }
}

// Norms on both sides: the state of the residual stream between two launches, x and the part whose result it still lacks.
static mix::PartNorm open_norm(const Decoder *d) {
    mix::PartNorm n{};
    n.mult = d->s.residual_mult;
    return n;
}
// Adds what is open, norms the sum for the next part; afterwards nothing is open.
template <class Fn>
static int32_t close_norm(Decoder *d, const mix::StepDesc &sd, mix::PartNorm &open, const float *pre, void *h, int pdl, Fn &&more) {
    mix::PartNorm n = open;
    n.x_out = n.x == d->x ? d->x_next : d->x, n.pre = pre, n.h = h;
    more(n);
    TRY(mix::launch_part_norm(d->f32, sd, residual(d, 0), n, nullptr, sd.rows, d->s.eps, d->s.width, d->ldw, d->ctx->sm_count, d->ctx->d_status,
                              n.x ? pdl : pdl & 2, d->ctx->stream));
    open = open_norm(d), open.x = n.x_out;
    return JGPT_OK;
}

static int32_t enqueue_layers(Decoder *d, Pool *p, const mix::StepDesc &sd, const std::vector<LatentBatch> &batches, uint64_t capture_rows) {
    const int W = d->s.width, R = sd.rows, ldw = d->ldw, eb = d->eb;
    const float eps = d->s.eps;
    cudaStream_t st = d->ctx->stream;
    int *status = d->ctx->d_status;
    const int pdl = d->overlap && !d->f32 && !capture_rows ? 3 : 0;
    const uint64_t slot = (uint64_t)d->R * W, mix_stride = (uint64_t)d->R * ldw;
    const bool deep = d->s.depth_average, after = d->s.norm_after, both = d->s.norm_both, gated_result = d->s.residual_gate;
    mix::PartNorm next = d->open = open_norm(d);
    const float res_scale = after ? d->s.residual_scale : 1.f;
    for (size_t i = 0; i < d->L.size(); i++) {
        DLayer &y = d->L[i];
        float *from = d->x, *to = deep ? d->slots + (i + 1) * slot : d->x;  // residual in front of the layer, its result
        uint8_t *rows_shifted = reinterpret_cast<uint8_t *>(d->h), *rows_plain = d->s.token_shift ? rows_shifted + mix_stride * eb : rows_shifted;
        void *layer_proj = y.v_source ? d->proj_first : d->proj;
        if (both) {
            TRY(close_norm(d, sd, next, y.n1w, rows_plain, pdl, [&](mix::PartNorm &n) {
                if (!d->s.token_shift) return;
                n.shifted = rows_shifted, n.share = y.share, n.state = p->state + y.shift_off, n.state_stride = p->state_stride, n.max_seqs = p->max_seqs;
            }));
        } else if (after) {  // the norms behind the sums leave h
            if (i == 0)
                TRY(mix::launch_residual_norm(d->f32, sd, residual(d, 0), nullptr, R, nullptr, eps, d->x, d->h, mix::ShiftArgs{}, W, ldw, status, pdl & 2, st));
        } else if (d->rms) {
            const DBranch *w = y.shift();
            mix::ShiftArgs sh{};
            if (w) {
                for (int k = 0; k < 5; k++) sh.mu[k] = w->mu + (size_t)k * W;
                sh.out_stride = mix_stride, sh.state = p->state + w->state_off + w->conv_off, sh.state_stride = p->state_stride, sh.max_seqs = p->max_seqs;
            }
            if (deep && i == 0) from = d->slots;
            TRY(mix::launch_residual_norm(d->f32, sd, residual(d, i), nullptr, R, y.n1w, eps, i == 0 || deep ? from : nullptr, d->h, sh, W, ldw, status,
                                          i == 0 ? pdl & 2 : pdl, st));
        } else if (i == 0) {
            TRY(mix::launch_embed(d->f32, sd, d->embed, ldw, d->pos, ldw, d->s.embed_scale,
                                  d->s.embed_norm ? mix::NormW{d->enw, d->enb} : mix::NormW{nullptr, nullptr}, mix::NormW{y.n1w, y.n1b}, eps, d->x,
                                  d->h, W, ldw, d->s.vocab, d->s.max_positions, status, pdl & 2, st));
        } else {
            TRY(mix::launch_layer_norm(d->f32, d->x, nullptr, mix::NormW{y.n1w, y.n1b}, eps, d->h, R, W, ldw, pdl, st));
        }
        if (const DBranch *w = y.shift()) {
            uint8_t *h = reinterpret_cast<uint8_t *>(d->h), *win = reinterpret_cast<uint8_t *>(y.w_in), *proj = reinterpret_cast<uint8_t *>(d->proj);
            const int hk = w->s.heads * w->DK;
            nt::Problem in[2] = {{h, win, proj, nullptr, R, 4 * hk, ldw, ldw, ldw, y.n_in, 1.f},
                                 {h + 4 * mix_stride * eb, win + (size_t)w->a1 * ldw * eb, proj + (size_t)w->a1 * eb, nullptr, R, w->ra, ldw, ldw, ldw, y.n_in, 1.f}};
            in[0].seg_n = hk, in[0].a_seg = (long long)mix_stride, in[1].act = nt::ACT_TANH;
            TRY(product(d, in, 2, nt::EPI_ACT, pdl));
        } else {
            nt::Problem in{d->h, y.w_in, layer_proj, nullptr, R, y.n_in, ldw, ldw, ldw, y.n_in, 1.f};
            in.bias = y.bias_in;
            if (gated_result && d->s.token_shift) in.seg_n = y.n_mix, in.a_seg = (long long)mix_stride, in.a_cap = 1;
            if (y.tanh_to) in.act = nt::ACT_TANH, in.act_from = y.tanh_from, in.act_to = y.tanh_to;
            TRY(product(d, &in, 1, y.tanh_to ? nt::EPI_ACT_SOME : nt::EPI_STORE, pdl));
        }
        for (DBranch &b : y.br) {
            if (b.s.kind == JGPT_MIX_ATTENTION) {
                mix::AttnArgs a{};
                a.proj = layer_proj, a.ldp = y.n_in, a.q_off = b.q, a.k_off = b.k, a.v_off = b.v, a.g_off = b.g;
                a.heads = b.s.heads, a.kv_heads = b.s.kv_heads, a.maps = b.maps, a.DK = b.DK, a.DV = b.DV, a.dim = b.s.dim, a.vdim = b.s.vdim;
                a.gate = b.s.gate, a.chunk = b.s.chunk, a.scale = b.s.score_scale, a.out_scale = b.s.out_scale;
                a.q_norm = b.q_norm, a.k_norm = b.k_norm, a.eps = eps, a.interleaved = b.s.rot_interleaved;
                if (b.rot >= 0) a.cs = d->rots[(size_t)b.rot].out, a.half = b.s.rot_dims / 2;
                a.whole_rows = b.s.qk_norm == JGPT_QK_NORM_ALL, a.row_inv = d->row_inv, a.window = b.s.window, a.keep = b.s.keep, a.sink = b.sink;
                if (const DBranch *f = b.v_first)
                    a.v_first = reinterpret_cast<uint8_t *>(d->proj_first) + (size_t)f->v * eb, a.ld_first = d->v_first_ld, a.vdim_first = f->s.vdim, a.DV_first = f->DV,
                    a.v_share = b.v_share;
                a.lambda = b.lambda, a.diff_scale = 1.f - b.s.diff;
                a.kv = p->vkv + p->vlayers[(size_t)b.kv_layer].offset, a.table = p->d_table, a.n_blocks = p->n_blocks, a.mbs = p->max_blocks_per_seq;
                a.out = d->mixed, a.ldo = y.n_out, a.out_off = b.out;
                a.sm_count = d->ctx->sm_count, a.status = status;
                TRY(mix::launch_attention(d->f32, sd, a, pdl, st));
            } else if (b.s.kind == JGPT_MIX_LATENT) {
                TRY(enqueue_latent(d, p, sd, batches, y, b, pdl));
            } else {
                uint8_t *proj = reinterpret_cast<uint8_t *>(d->proj), *z = reinterpret_cast<uint8_t *>(d->z);
                nt::Problem zp[2];
                int nz = 0;
                if (b.a1 >= 0)
                    zp[nz++] = nt::Problem{proj + (size_t)b.a1 * eb, b.w_a2, z + (size_t)b.za * eb, nullptr, R, b.s.heads * b.DK, b.ra, y.n_in, b.ra, y.n_z, 1.f};
                if (b.g1 >= 0)
                    zp[nz++] = nt::Problem{proj + (size_t)b.g1 * eb, b.w_g2, z + (size_t)b.zg * eb, nullptr, R, b.s.heads * b.DV, b.rg, y.n_in, b.rg, y.n_z, 1.f};
                if (nz) TRY(product(d, zp, nz, nt::EPI_STORE, pdl));
                mix::RecArgs a = rec_args(b);
                a.proj = d->proj, a.ldp = y.n_in, a.z = d->z, a.ldz = y.n_z, a.eps = eps;
                if (b.s.kind == JGPT_MIX_HGRN2) a.z = d->proj, a.ldz = y.n_in;
                a.state = p->state + b.state_off, a.state_stride = p->state_stride, a.max_seqs = p->max_seqs;
                a.out = d->mixed, a.ldo = y.n_out, a.raw = d->raw, a.chunk_ws = d->chunk_ws, a.chunk_ws_floats = d->chunk_ws_floats, a.sm_count = d->ctx->sm_count, a.status = status;
                TRY(mix::launch_recurrent(d->f32, sd, a, pdl, st));
            }
        }
        if (both) {
            nt::Problem out{d->mixed, y.w_out, d->y, nullptr, R, ldw, y.n_out, y.n_out, y.n_out, ldw, 1.f};
            TRY(product(d, &out, 1, nt::EPI_STORE, pdl));
            next.y = d->y, next.post = y.post1;
            if (gated_result) next.gate = reinterpret_cast<uint8_t *>(layer_proj) + (size_t)y.n_mix * eb, next.ldg = y.n_in;
            if (y.ff) {
                TRY(close_norm(d, sd, next, y.n2w, d->h, pdl, [](mix::PartNorm &) {}));
                const bool one = y.ff_kind == JGPT_FF_XIELU || y.ff_kind == JGPT_FF_RELU2;
                const int n_act = one ? y.n_up : y.ffp;
                nt::Problem in{d->h, y.w_gu, d->act, nullptr, R, one ? y.n_up : 2 * y.ffp, ldw, ldw, ldw, n_act, 1.f};
                set_activation(y, in);
                in.act_to = y.ffp, in.bias = y.bias_up;
                TRY(product(d, &in, 1, !one ? nt::EPI_GATE : gated_result ? nt::EPI_ACT_SOME : nt::EPI_ACT, pdl));
                nt::Problem down{d->act, y.w_down, d->y, nullptr, R, ldw, y.ffp, n_act, y.ffp, ldw, 1.f};
                TRY(product(d, &down, 1, nt::EPI_STORE, pdl));
                next.y = d->y, next.post = y.post2;
                if (gated_result) next.gate = reinterpret_cast<uint8_t *>(d->act) + (size_t)y.ffp * eb, next.ldg = n_act;
            }
            d->open = next;
            if (capture_rows) {  // the sum as it will be formed in front of the next part
                mix::PartNorm n = next;
                n.x_out = next.x == d->x ? d->x_next : d->x;
                TRY(mix::launch_part_norm(d->f32, sd, residual(d, 0), n, nullptr, R, eps, W, ldw, d->ctx->sm_count, status, 0, st));
                JGPT_CUDA_TRY(cudaMemcpy2DAsync(d->capture + (uint64_t)i * capture_rows * W, sizeof(float) * W, n.x_out, sizeof(float) * ldw, sizeof(float) * W, capture_rows,
                                                cudaMemcpyDeviceToHost, st));
            }
            continue;
        }
        nt::Problem out{d->mixed, y.w_out, to, nullptr, R, W, y.n_out, y.n_out, y.n_out, W, 1.f};
        out.res = from, out.colscale = y.ls1, out.res_scale = res_scale;
        TRY(product(d, &out, 1, nt::EPI_ADD_F32, pdl));
        if (after) TRY(mix::launch_post_norm(d->f32, d->x, R, y.n1w, eps, d->h, mix::MoeSum{}, W, ldw, pdl, st));
        mix::MoeSum moe{};
        if (y.effp) {
            TRY(enqueue_moe(d, y, R, pdl, moe));
        } else if (y.ff) {
            if (d->rms && !after) {
                mix::RowSource src{};
                src.slots = to, src.n_slots = 1;
                TRY(mix::launch_residual_norm(d->f32, sd, src, nullptr, R, y.n2w, eps, nullptr, d->h, mix::ShiftArgs{}, W, ldw, status, pdl, st));
            } else if (!after) {
                TRY(mix::launch_layer_norm(d->f32, d->x, nullptr, mix::NormW{y.n2w, y.n2b}, eps, d->h, R, W, ldw, pdl, st));
            }
            const bool gated = y.ff_kind != JGPT_FF_XIELU && y.ff_kind != JGPT_FF_RELU2;
            nt::Problem gu{d->h, y.w_gu, d->act, nullptr, R, gated ? 2 * y.ffp : y.ffp, ldw, ldw, ldw, y.ffp, 1.f};
            set_activation(y, gu);
            TRY(product(d, &gu, 1, gated ? nt::EPI_GATE : nt::EPI_ACT, pdl));
            nt::Problem down{d->act, y.w_down, to, nullptr, R, W, y.ffp, y.ffp, y.ffp, W, 1.f};
            down.colscale = y.ls2, down.res_scale = res_scale;
            TRY(product(d, &down, 1, nt::EPI_ADD_F32, pdl));
        }
        if (after && y.ff) TRY(mix::launch_post_norm(d->f32, d->x, R, y.n2w, eps, d->h, moe, W, ldw, pdl, st));
        if (capture_rows) {
            if (deep) TRY(mix::launch_residual_norm(d->f32, sd, residual(d, i + 1), nullptr, R, d->fnw, eps, d->x, nullptr, mix::ShiftArgs{}, W, ldw, status, 0, st));
            JGPT_CUDA_TRY(cudaMemcpyAsync(d->capture + (uint64_t)i * capture_rows * W, d->x, sizeof(float) * capture_rows * W, cudaMemcpyDeviceToHost, st));
        }
    }
    return JGPT_OK;
}

// Final norm, logits and token choice of wanted rows [w0, w0 + n).
static int32_t enqueue_head(Decoder *d, const mix::StepDesc &sd, int w0, int n, bool pick, const SampleSpec &spec) {
    cudaStream_t st = d->ctx->stream;
    const int pdl = d->overlap && !d->f32 && w0 == 0 ? 3 : 0;
    if (d->s.norm_both) {
        mix::PartNorm last = d->open;
        last.pre = d->fnw, last.h = d->h;
        TRY(mix::launch_part_norm(d->f32, sd, residual(d, 0), last, sd.want + w0, n, d->s.eps, d->s.width, d->ldw, d->ctx->sm_count, d->ctx->d_status, pdl, st));
    } else if (d->rms)
        TRY(mix::launch_residual_norm(d->f32, sd, residual(d, d->L.size()), sd.want + w0, n, d->fnw, d->s.eps, nullptr, d->h, mix::ShiftArgs{}, d->s.width,
                                      d->ldw, d->ctx->d_status, pdl, st));
    else TRY(mix::launch_layer_norm(d->f32, d->x, sd.want + w0, mix::NormW{d->fnw, d->fnb}, d->s.eps, d->h, n, d->s.width, d->ldw, pdl, st));
    nt::Problem p{d->h, d->head ? d->head : d->embed, d->logits, nullptr, n, d->s.vocab, d->ldw, d->ldw, d->ldw, d->s.vocab, d->s.logit_scale};
    TRY(product(d, &p, 1, nt::EPI_SCALE_F32, pdl & 1));
    if (!pick) return JGPT_OK;
    if (spec.temperature > 0.f) return launch_sample(d->logits, d->samp, n, d->s.vocab, spec, d->d_u + w0, d->d_next + w0, st);
    return launch_argmax(d->logits, n, d->s.vocab, d->d_next + w0, st);
}

// Replays the step's graph, captures it at the second step of its kind, or runs the launches one by one.
template <class Fn>
static int32_t run_graph(Decoder *d, const Pool *p, int n, int bucket, Fn &&enqueue) {
    cudaStream_t st = d->ctx->stream;
    for (Decoder::Graph &g : d->graphs) {
        if (g.pool != p || g.generation != p->generation || g.n != n || g.bucket != bucket) continue;
        g.last_use = ++d->graph_clock;
        if (!g.exec && !g.failed) {
            cudaGraph_t graph = nullptr;
            JGPT_CUDA_TRY(cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal));
            const int32_t rc = enqueue();
            const cudaError_t e = cudaStreamEndCapture(st, &graph);
            if (rc || e != cudaSuccess || cudaGraphInstantiate(&g.exec, graph, 0) != cudaSuccess) g.exec = nullptr, g.failed = true;
            if (graph) cudaGraphDestroy(graph);
            cudaGetLastError();
        }
        if (!g.exec) break;
        JGPT_CUDA_TRY(cudaGraphLaunch(g.exec, st));
        return JGPT_OK;
    }
    bool known = false;
    for (const Decoder::Graph &g : d->graphs) known = known || (g.pool == p && g.generation == p->generation && g.n == n && g.bucket == bucket);
    if (!known) {
        if (d->graphs.size() >= 64) {  // forget the one that has not been used for longest
            auto old = std::min_element(d->graphs.begin(), d->graphs.end(), [](const Decoder::Graph &x, const Decoder::Graph &y) { return x.last_use < y.last_use; });
            if (old->exec) cudaGraphExecDestroy(old->exec);
            d->graphs.erase(old);
        }
        Decoder::Graph g;
        g.pool = p, g.generation = p->generation, g.n = n, g.bucket = bucket, g.last_use = ++d->graph_clock;
        d->graphs.push_back(g);
    }
    return enqueue();
}

int32_t decoder_step(Decoder *d, Pool *p, jgpt_kvpool poolh, const StepCall &c) {
    TRY(decoder_check_pool(d, p));
    JGPT_CUDA_TRY(make_current(d->ctx));
    TRY(missing_weights(d));
    JGPT_REQUIRE(c.n >= 1 && c.seq_ids && c.starts && c.ids && c.starts[0] == 0, JGPT_ERR_INVALID_ARGUMENT, "null pointer or empty step");
    const int rows = c.starts[c.n];
    JGPT_REQUIRE(rows >= c.n && rows <= d->R, JGPT_ERR_INVALID_ARGUMENT, "a step of %d rows; the model's workspace holds %d", rows, d->R);
    JGPT_REQUIRE(c.n_want >= 0 && (c.n_want == 0 || c.want), JGPT_ERR_INVALID_ARGUMENT, "null list of wanted rows");
    JGPT_REQUIRE(c.spec.temperature <= 0.f || c.u01 || c.n_want == 0, JGPT_ERR_INVALID_ARGUMENT, "sampling needs one draw per row");
    for (int i = 0; i < c.n_want; i++)
        JGPT_REQUIRE(c.want[i] >= 0 && c.want[i] < rows, JGPT_ERR_OUT_OF_RANGE, "wanted row %d of %d", c.want[i], rows);
    for (int i = 0; i < rows; i++)
        JGPT_REQUIRE(c.ids[i] >= 0 && c.ids[i] < d->s.vocab, JGPT_ERR_OUT_OF_RANGE, "token id %d outside [0,%d)", c.ids[i], d->s.vocab);
    std::vector<char> seen((size_t)p->max_seqs, 0);
    int n_tiles = 0, n_single = 0;
    for (int i = 0; i < c.n; i++) {
        const int s = c.seq_ids[i], T = c.starts[i + 1] - c.starts[i];
        JGPT_REQUIRE(s >= 0 && s < p->max_seqs && p->seqs[(size_t)s].used, JGPT_ERR_OUT_OF_RANGE, "sequence %d is not allocated", s);
        JGPT_REQUIRE(T >= 1 && !seen[(size_t)s], JGPT_ERR_INVALID_ARGUMENT, "entry %d: no tokens, or its sequence appears twice", i);
        seen[(size_t)s] = 1;
        JGPT_REQUIRE(p->seqs[(size_t)s].len + T <= d->s.max_positions, JGPT_ERR_ILLEGAL_STATE, "sequence %d: %d + %d tokens exceed the %d positions", s,
                     p->seqs[(size_t)s].len, T, d->s.max_positions);
    }
    JGPT_REQUIRE(c.n_want <= d->R, JGPT_ERR_INVALID_ARGUMENT, "%d wanted rows; the workspace holds %d", c.n_want, d->R);
    // blocks for every entry, or none
    for (int i = 0; i < c.n; i++) {
        const int s = c.seq_ids[i], T = c.starts[i + 1] - c.starts[i];
        const int32_t rc = jgpt_seq_reserve(poolh, s, p->seqs[(size_t)s].len + T);
        if (rc) {
            const std::string keep = last_error_ref();
            for (int j = 0; j < i; j++) pool_trim_reservation(p, c.seq_ids[j], p->seqs[(size_t)c.seq_ids[j]].len);
            last_error_ref() = keep;
            return rc;
        }
    }
    // ---- descriptors ----
    int *hd = d->h_desc;
    size_t at = 0;
    auto take = [&](size_t n) {
        const size_t o = at;
        at += (n + 3) / 4 * 4;
        return o;
    };
    const size_t o_tok = take((size_t)rows), o_pos = take((size_t)rows), o_seq = take((size_t)rows), o_seg = take(6 * (size_t)c.n);
    const size_t o_ent = take((size_t)rows), o_lat_single = take(6 * (size_t)c.n), o_lat_short = take(6 * (size_t)c.n), o_lat_long = take(4 * (size_t)c.n);
    const size_t o_single = take((size_t)c.n), o_short = take((size_t)c.n), o_want = take((size_t)c.n_want), o_long = take(2 * (size_t)c.n);
    int max_len = 0, n_short = 0, n_long = 0, n_chunks = 0;
    const int long_min = d->long_min;
    mix::Seg *segs = reinterpret_cast<mix::Seg *>(hd + o_seg);
    for (int i = 0; i < c.n; i++) {
        const int s = c.seq_ids[i], r0 = c.starts[i], T = c.starts[i + 1] - r0;
        const SeqState &ss = p->seqs[(size_t)s];
        segs[i] = mix::Seg{s, r0, T, ss.len, ss.conv_set, 0};
        max_len = std::max(max_len, ss.len + T);
        for (int t = 0; t < T; t++) hd[o_tok + r0 + t] = c.ids[r0 + t], hd[o_pos + r0 + t] = ss.len + t, hd[o_seq + r0 + t] = s, hd[o_ent + r0 + t] = i;
        if (T == 1) hd[o_single + n_single++] = i;
        if (long_min == 0 || T < long_min) hd[o_short + n_short++] = i;
        else {
            hd[o_long + 2 * n_long] = i, hd[o_long + 2 * n_long + 1] = n_chunks, n_long++;
            n_chunks += (T + mix::kRecChunk - 1) / mix::kRecChunk;
        }
    }
    for (int i = 0; i < c.n_want; i++) hd[o_want + i] = c.want[i];
    const size_t o_chunk = take(2 * (size_t)n_chunks), o_tile = at;
    for (int l = 0, k = 0; l < n_long; l++) {
        const int i = hd[o_long + 2 * l], T = c.starts[i + 1] - c.starts[i];
        for (int t = 0; t < T; t += mix::kRecChunk, k++) hd[o_chunk + 2 * k] = i, hd[o_chunk + 2 * k + 1] = t;
    }
    // query tiles: the same list serves every layer, so tiles hold as many tokens as the layer with the largest groups allows
    int qt = 64;
    for (const DLayer &y : d->L)
        for (const DBranch &b : y.br)
            if (b.s.kind == JGPT_MIX_ATTENTION) qt = std::min(qt, mix::attn_query_tile(b.s.heads, b.s.kv_heads));
    for (int i = 0; i < c.n; i++) {
        const int T = c.starts[i + 1] - c.starts[i];
        if (T > 1)
            for (int t = 0; t < T; t += qt) hd[o_tile + 2 * n_tiles] = i, hd[o_tile + 2 * n_tiles + 1] = t, n_tiles++;
    }
    at = o_tile;
    take(2 * (size_t)n_tiles);
    // latent attention: long entries in batches that fit the workspace, with tiles of query tokens of their own; the others'
    // rows as one range (running tokens and short portions lie together in what the scheduler sends)
    mix::StepDesc sd{};
    std::vector<LatentBatch> batches;
    const size_t o_lat_tile = at;
    int n_lat_long = 0, n_lat_tiles = 0;
    sd.lat_lo = rows;
    mix::LatentEntry *lat_long = reinterpret_cast<mix::LatentEntry *>(hd + o_lat_long);
    mix::Seg *lat_single = reinterpret_cast<mix::Seg *>(hd + o_lat_single), *lat_short = reinterpret_cast<mix::Seg *>(hd + o_lat_short);
    int n_lat_single = 0;
    for (int i = 0; d->cq && i < c.n; i++) {
        const int T = segs[i].T, pos0 = segs[i].pos0, back = d->max_window > 0 ? std::min(pos0, d->max_window - 1) : pos0;
        if (d->lat_min == 0 || T < std::max(d->lat_min, 2) || (long long)back + T > d->kvx_rows) {
            sd.lat_lo = std::min(sd.lat_lo, segs[i].row0), sd.lat_hi = segs[i].row0 + T;
            if (T > 1) lat_short[sd.n_lat_short++] = segs[i], sd.lat_short_max = std::max(sd.lat_short_max, T);
            else lat_single[n_lat_single++] = segs[i];
            continue;
        }
        if (batches.empty() || batches.back().rows + back + T > d->kvx_rows) batches.push_back(LatentBatch{n_lat_long, 0, 0, 0, n_lat_tiles, 0});
        LatentBatch &g = batches.back();
        lat_long[n_lat_long] = mix::LatentEntry{i, pos0 - back, back + T, g.rows};
        for (int t = 0; t < T; t += mix::kLatentTile, g.n_tiles++)
            hd[o_lat_tile + 2 * n_lat_tiles] = n_lat_long, hd[o_lat_tile + 2 * n_lat_tiles + 1] = t, n_lat_tiles++;
        g.n++, g.rows += back + T, g.max_keys = std::max(g.max_keys, back + T), n_lat_long++;
    }
    at = o_lat_tile + 2 * (size_t)n_lat_tiles;
    JGPT_REQUIRE(at <= desc_ints(d), JGPT_ERR_INVALID_ARGUMENT, "step descriptors need %zu words, there are %zu", at, desc_ints(d));
    cudaStream_t st = d->ctx->stream;
    const int *dd = d->d_desc;
    sd.tok = dd + o_tok, sd.pos = dd + o_pos, sd.seq = dd + o_seq, sd.segs = reinterpret_cast<const mix::Seg *>(dd + o_seg);
    sd.tiles = reinterpret_cast<const int2 *>(dd + o_tile), sd.singles = dd + o_single, sd.want = dd + o_want;
    sd.ent = dd + o_ent, sd.lat_singles = reinterpret_cast<const mix::Seg *>(dd + o_lat_single), sd.lat_short = reinterpret_cast<const mix::Seg *>(dd + o_lat_short), sd.lat_long = reinterpret_cast<const mix::LatentEntry *>(dd + o_lat_long);
    sd.lat_tiles = reinterpret_cast<const int2 *>(dd + o_lat_tile);
    sd.rows = rows, sd.n_segs = c.n, sd.n_tiles = n_tiles, sd.n_singles = n_single, sd.n_want = c.n_want, sd.max_len = max_len;
    sd.qt = qt;
    sd.short_segs = dd + o_short, sd.long_segs = reinterpret_cast<const int2 *>(dd + o_long), sd.chunks = reinterpret_cast<const int2 *>(dd + o_chunk);
    sd.n_short = n_short, sd.n_long = n_long, sd.n_chunks = n_chunks;

    if (n_tiles == 0) sd.max_len = std::min(up(max_len, 256), d->s.max_positions);  // a bucket: it only shapes the launches
    uint64_t cap_rows = 0;
    if (d->capture) {
        JGPT_REQUIRE(d->capture_floats >= (uint64_t)d->L.size() * rows * d->s.width, JGPT_ERR_INVALID_ARGUMENT, "capture buffer is too small");
        cap_rows = (uint64_t)rows;
    }
    float *capture_to = d->capture;
    const bool pick = c.next_host != nullptr;
    if (pick && c.spec.temperature > 0.f && c.n_want) {
        if (!d->samp) TRY(dalloc(d, (void **)&d->samp, sizeof(float) * (uint64_t)d->logit_rows * d->s.vocab));
        std::copy(c.u01, c.u01 + c.n_want, d->h_u);
        JGPT_CUDA_TRY(cudaMemcpyAsync(d->d_u, d->h_u, sizeof(float) * c.n_want, cudaMemcpyHostToDevice, st));
    }
    auto enqueue = [&]() -> int32_t {
        JGPT_CUDA_TRY(cudaMemcpyAsync(d->d_desc, hd, sizeof(int) * at, cudaMemcpyHostToDevice, st));
        TRY(enqueue_layers(d, p, sd, batches, cap_rows));
        for (int w0 = 0; w0 < c.n_want; w0 += d->logit_rows) {
            const int n = std::min(d->logit_rows, c.n_want - w0);
            TRY(enqueue_head(d, sd, w0, n, pick, c.spec));
            if (c.logits_host)
                JGPT_CUDA_TRY(cudaMemcpyAsync(c.logits_host + (size_t)w0 * d->s.vocab, d->logits, sizeof(float) * (size_t)n * d->s.vocab,
                                              cudaMemcpyDeviceToHost, st));
        }
        if (pick && c.n_want) JGPT_CUDA_TRY(cudaMemcpyAsync(d->h_next, d->d_next, sizeof(int) * c.n_want, cudaMemcpyDeviceToHost, st));
        JGPT_CUDA_TRY(status_enqueue_read(d->ctx));
        return JGPT_OK;
    };
    bool plain = d->use_graphs && n_tiles == 0 && pick && !c.logits_host && !capture_to && c.spec.temperature <= 0.f && c.n_want == c.n;
    for (int i = 0; plain && i < c.n; i++) plain = c.want[i] == i;
    d->capture = nullptr;
    if (plain) TRY(run_graph(d, p, c.n, sd.max_len, enqueue));
    else {
        d->capture = capture_to;
        const int32_t rc = enqueue();
        d->capture = nullptr;
        if (rc) return rc;
    }
    JGPT_CUDA_TRY(cudaStreamSynchronize(st));
    TRY(status_check_after_sync(d->ctx, p, "forward step"));
    if (pick) std::copy(d->h_next, d->h_next + c.n_want, c.next_host);
    for (int i = 0; i < c.n; i++) {
        SeqState &ss = p->seqs[(size_t)c.seq_ids[i]];
        ss.len += c.starts[i + 1] - c.starts[i];
        ss.conv_set ^= 1;
        ss.tick = ++p->clock;
    }
    return JGPT_OK;
}

// ------------------------------------------------------------------------------------------------
// The fixed-block model's forms
// ------------------------------------------------------------------------------------------------
int32_t decoder_prefill_batch(Decoder *d, jgpt_kvpool poolh, const int *seq_ids, const int *starts, const int *ids, const int *rope_offsets,
                              int n, float *all_logits, float *last_logits, int *next) {
    Pool *p = pool_registry().get(poolh);
    TRY(decoder_check_pool(d, p));
    JGPT_REQUIRE(n >= 1 && seq_ids && starts && ids && rope_offsets, JGPT_ERR_INVALID_ARGUMENT, "null pointer or empty batch");
    JGPT_REQUIRE(!all_logits || n == 1, JGPT_ERR_INVALID_ARGUMENT, "all-row logits are available for one sequence at a time");
    for (int i = 0; i < n; i++) {
        JGPT_REQUIRE(rope_offsets[i] == 0, JGPT_ERR_UNSUPPORTED, "positions of a layered decoder start at 0");
        const int s = seq_ids[i];
        JGPT_REQUIRE(s >= 0 && s < p->max_seqs && p->seqs[(size_t)s].used, JGPT_ERR_OUT_OF_RANGE, "sequence %d is not allocated", s);
        p->seqs[(size_t)s].len = 0;  // a prefill starts the sequence over
    }
    std::vector<int> want;
    if (all_logits)
        for (int r = 0; r < starts[n]; r++) want.push_back(r);
    else
        for (int i = 0; i < n; i++) want.push_back(starts[i + 1] - 1);
    StepCall c;
    c.n = n, c.seq_ids = seq_ids, c.starts = starts, c.ids = ids, c.n_want = (int)want.size(), c.want = want.data();
    c.logits_host = all_logits ? all_logits : last_logits;
    std::vector<int> picked(want.size());
    if (next) c.next_host = picked.data();
    TRY(decoder_step(d, p, poolh, c));
    if (all_logits && last_logits) std::copy(all_logits + (size_t)(starts[n] - 1) * d->s.vocab, all_logits + (size_t)starts[n] * d->s.vocab, last_logits);
    if (next) {
        if (all_logits) next[0] = picked.back();
        else std::copy(picked.begin(), picked.end(), next);
    }
    return JGPT_OK;
}

int32_t decoder_decode(Decoder *d, jgpt_kvpool poolh, const int *seq_ids, const int *ids, const int *len_before, const int *rope_pos, int n,
                       float *logits, int *next, const SampleSpec &spec, const float *u01) {
    Pool *p = pool_registry().get(poolh);
    TRY(decoder_check_pool(d, p));
    JGPT_REQUIRE(n >= 1 && seq_ids && ids && len_before && rope_pos, JGPT_ERR_INVALID_ARGUMENT, "null pointer or empty batch");
    std::vector<int> starts((size_t)n + 1), want((size_t)n);
    for (int i = 0; i < n; i++) {
        const int s = seq_ids[i];
        JGPT_REQUIRE(s >= 0 && s < p->max_seqs && p->seqs[(size_t)s].used, JGPT_ERR_OUT_OF_RANGE, "sequence %d is not allocated", s);
        JGPT_REQUIRE(p->seqs[(size_t)s].len == len_before[i], JGPT_ERR_ILLEGAL_STATE, "sequence %d holds %d tokens, the call says %d", s,
                     p->seqs[(size_t)s].len, len_before[i]);
        JGPT_REQUIRE(rope_pos[i] == len_before[i], JGPT_ERR_INVALID_ARGUMENT, "positions of a layered decoder follow the length");
        starts[(size_t)i + 1] = i + 1, want[(size_t)i] = i;
    }
    StepCall c;
    c.n = n, c.seq_ids = seq_ids, c.starts = starts.data(), c.ids = ids, c.n_want = n, c.want = want.data();
    c.logits_host = logits, c.next_host = next, c.spec = spec, c.u01 = u01;
    return decoder_step(d, p, poolh, c);
}

int32_t decoder_generate_greedy(Decoder *d, jgpt_kvpool poolh, const int *prompt, int S, int max_new, int *out, int *n_sampled) {
    Pool *p = pool_registry().get(poolh);
    TRY(decoder_check_pool(d, p));
    JGPT_REQUIRE(prompt && out && S >= 1 && max_new >= 0, JGPT_ERR_INVALID_ARGUMENT, "bad prompt");
    JGPT_REQUIRE(S + std::max(max_new, 1) - 1 <= d->s.max_positions, JGPT_ERR_INVALID_ARGUMENT, "prompt %d + %d new tokens exceed the %d positions", S,
                 max_new, d->s.max_positions);
    std::copy(prompt, prompt + S, out);
    std::fill(out + S, out + S + max_new, 0);
    if (n_sampled) *n_sampled = 0;
    if (max_new == 0) return JGPT_OK;
    int32_t seq = -1;
    TRY(jgpt_seq_alloc(poolh, &seq));
    const int32_t rc = [&]() -> int32_t {
        int tok = 0;
        for (int t0 = 0; t0 < S; t0 += d->R) {  // the prompt in portions of the workspace's rows
            const int T = std::min(d->R, S - t0), starts[2] = {0, T}, last = T - 1;
            StepCall c;
            c.n = 1, c.seq_ids = &seq, c.starts = starts, c.ids = prompt + t0;
            if (t0 + T == S) c.n_want = 1, c.want = &last, c.next_host = &tok;
            TRY(decoder_step(d, p, poolh, c));
        }
        for (int j = 0;; j++) {
            out[S + j] = tok;
            if (n_sampled) *n_sampled = j + 1;
            if (tok == 0 || j + 1 == max_new) return JGPT_OK;
            const int len = S + j;
            TRY(decoder_decode(d, poolh, &seq, &tok, &len, &len, 1, nullptr, &tok, SampleSpec(), nullptr));
        }
    }();
    const std::string keep = last_error_ref();
    jgpt_seq_free(poolh, seq);
    last_error_ref() = keep;
    return rc;
}

}  // namespace jgpt

using namespace jgpt;

#define GET_DECODER(d, h)                                                   \
    Decoder *d = decoder_registry().get(h);                                 \
    JGPT_REQUIRE(d, JGPT_ERR_BAD_HANDLE, "not a layered decoder's handle"); \
    JGPT_CUDA_TRY(make_current(d->ctx))

extern "C" {

int32_t jgpt_decoder_create(jgpt_ctx ctxh, const jgpt_decoder_spec *spec, const jgpt_layer_spec *layers, int32_t dtype, int32_t max_rows,
                            jgpt_model *out) {
    Ctx *c = ctx_registry().get(ctxh);
    JGPT_REQUIRE(c, JGPT_ERR_BAD_HANDLE, "bad context handle");
    JGPT_REQUIRE(spec && layers && out, JGPT_ERR_INVALID_ARGUMENT, "null pointer");
    JGPT_REQUIRE(spec->vocab > 0 && spec->width > 0 && spec->max_positions > 0 && spec->n_layers > 0 && max_rows > 0, JGPT_ERR_INVALID_ARGUMENT,
                 "model dimensions must be positive");
    const bool rms = spec->norm == JGPT_NORM_RMS;
    JGPT_REQUIRE(rms || spec->norm == JGPT_NORM_LAYER, JGPT_ERR_UNSUPPORTED, "norm %d", spec->norm);
    JGPT_REQUIRE(rms ? !spec->pos_table && !spec->embed_norm : !spec->layer_scale && !spec->depth_average && spec->residual_mult == 1.f, JGPT_ERR_UNSUPPORTED,
                 "layer norms go with embedding norms and learned positions, RMS norms with residual factors and depth averages");
    JGPT_REQUIRE(!spec->norm_after || (rms && !spec->layer_scale && !spec->depth_average && spec->residual_mult == 1.f), JGPT_ERR_UNSUPPORTED,
                 "norms behind the sums are RMS norms over a plain residual");
    JGPT_REQUIRE(!spec->norm_both || (rms && !spec->norm_after && !spec->layer_scale && !spec->depth_average), JGPT_ERR_UNSUPPORTED,
                 "norms on both sides are RMS norms without layer scales and depth averages");
    JGPT_REQUIRE(spec->norm_both || (!spec->token_shift && !spec->residual_gate), JGPT_ERR_UNSUPPORTED, "token shifts and gated results go with norms on both sides");
    JGPT_REQUIRE(dtype == JGPT_DTYPE_BF16 || dtype == JGPT_DTYPE_F32, JGPT_ERR_INVALID_ARGUMENT, "dtype %d", dtype);
    JGPT_CUDA_TRY(make_current(c));
    Decoder *d = new Decoder();
    d->use_graphs = env_int("JGPT_B200_DECODE_GRAPH", 1), d->overlap = env_int("JGPT_B200_STEP_OVERLAP", 1);
    d->ctx = c, d->s = *spec, d->f32 = dtype == JGPT_DTYPE_F32, d->eb = d->f32 ? 4 : 2, d->R = max_rows, d->ldw = up(spec->width, 8);
    const int32_t rc = build(d, layers);
    if (rc) {
        const std::string keep = last_error_ref();
        release(d);
        last_error_ref() = keep;
        return rc;
    }
    *out = decoder_registry().add(d);
    return JGPT_OK;
}

int32_t jgpt_decoder_set_tensor(jgpt_model h, int32_t layer, int32_t branch, int32_t role, const float *host, int32_t rows, int32_t cols) {
    GET_DECODER(d, h);
    JGPT_REQUIRE(layer >= -1 && layer < (int)d->L.size(), JGPT_ERR_OUT_OF_RANGE, "layer %d outside [-1,%zu)", layer, d->L.size());
    JGPT_REQUIRE(host && rows >= 1 && cols >= 1, JGPT_ERR_INVALID_ARGUMENT, "null or empty tensor");
    return set_tensor(d, layer, branch, role, host, rows, cols);
}

int32_t jgpt_decoder_capture_layers(jgpt_model h, float *host, uint64_t n_floats) {
    GET_DECODER(d, h);
    d->capture = host, d->capture_floats = host ? n_floats : 0;
    return JGPT_OK;
}

int32_t jgpt_decoder_new_pool(jgpt_model h, int32_t n_blocks, int32_t max_seqs, int32_t max_blocks_per_seq, jgpt_kvpool *out) {
    GET_DECODER(d, h);
    JGPT_REQUIRE(out, JGPT_ERR_INVALID_ARGUMENT, "out is null");
    return pool_create_layered(d->ctx, d->kv, d->eb, n_blocks, max_seqs, max_blocks_per_seq, d->state_stride, out);
}

int32_t jgpt_forward_step(jgpt_model h, jgpt_kvpool poolh, int32_t n, const int32_t *seq_ids_host, const int32_t *starts_host,
                          const int32_t *ids_host, int32_t n_want, const int32_t *want_rows_host, float *logits_host, int32_t *next_tokens_host) {
    GET_DECODER(d, h);
    StepCall c;
    c.n = n, c.seq_ids = seq_ids_host, c.starts = starts_host, c.ids = ids_host, c.n_want = n_want, c.want = want_rows_host;
    c.logits_host = logits_host, c.next_host = next_tokens_host;
    return decoder_step(d, pool_registry().get(poolh), poolh, c);
}

}  // extern "C"
