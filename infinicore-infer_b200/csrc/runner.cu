// The native step: replays a model's launch records (runner.h) for one batch.
//
// One call launches every kernel of a run of records (for the standard stack: the whole step, embedding to logits)
// where Python would make a dozen calls a layer.  Which kernel runs a record is decided here and nowhere else:
//
//   float32       every product on the CUDA cores (gemm_f32, no tensor cores), attention by the row kernel
//   bfloat16      products by the rules of host_rules.h (jk::product_route):
//                   rows <= 16          the weight-streaming kernels of linear_small.cu (q/k/v with rotation and cache
//                                       write in the epilogue, gate/up with SwiGLU in the epilogue)
//                   few rows, wide      the tcgen05 kernel with the weights on the MMA's M side (gemm_skinny.cu)
//                   many rows, wide     the tiled tcgen05 kernel (q/k/v epilogue, SwiGLU epilogue, residual add by TMA)
//                   else                cuBLAS, bfloat16 operands, float32 accumulation and output, with the rotary
//                                       kernel, the SwiGLU kernel and the fused add + norm kernel around it
//                 attention: tiles of requests with many rows -> attention_tcgen05 (or the mma.sync kernel);
//                            rows of requests with few rows -> the split-key decode kernel
//   steps of at most 16 rows run without norm kernels where three records in a row allow it (a product that adds into
//   the stream, a norm, the product after it): see fuse_norm below.
//
// The kernels live in their own shared objects; the caller hands their entry points over once (jk_runner_bind).
// Nothing is allocated here.
#include "common.cuh"
#include "runner.h"

#include <cublas_v2.h>
#include <cstdlib>
#include <mutex>

JK_DEFINE_ERROR_BUFFER(jk_runner)

static RunnerFns g_fns = {};
static bool g_bound = false;
JK_EXPORT const RunnerFns *jk_runner_fns() { return g_bound ? &g_fns : nullptr; }

JK_EXPORT int jk_runner_bind(const RunnerFns *fns) {
    JK_REQUIRE(fns != nullptr, "runner_bind: no table");
    // a table adds to what is bound already (two users of this library in one process may need different modules): an
    // entry that this caller leaves empty keeps what an earlier caller gave
    static_assert(sizeof(RunnerFns) % sizeof(void *) == 0, "the table is a list of pointers");
    void *const *from = (void *const *)fns;
    void **to = (void **)&g_fns;
    for (size_t i = 0; i < sizeof(RunnerFns) / sizeof(void *); ++i)
        if (from[i] != nullptr) to[i] = from[i];
    // the tcgen05 modules may be left out by a caller whose model or step size never reaches them (they are then not
    // even compiled); everything else is needed by every model
    const RunnerFns &f = g_fns;
    JK_REQUIRE(f.embed && f.add_rmsnorm && f.residual_add && f.swiglu && f.rope_kv && f.gemm_f32 && f.linear_small &&
               f.linear_small_qkv && f.linear_small_supports && f.linear_small_qkv_supports && f.linear_small_norm_supports &&
               f.linear_small_norm && f.linear_small_qkv_norm && f.attention_rows && f.attention_decode && f.attention_prefill &&
               f.attention_prefill_supports && f.err_elementwise && f.err_linear_small && f.err_attention,
               "runner_bind: an entry that every model needs is empty");
    JK_REQUIRE((f.gemm_tcgen05 != nullptr) == (f.gemm_tcgen05_qkv != nullptr) && (f.gemm_tcgen05 != nullptr) == (f.gemm_skinny != nullptr) &&
               (f.gemm_tcgen05 != nullptr) == (f.err_gemm_tcgen05 != nullptr) &&
               (f.attention_tcgen05 != nullptr) == (f.err_attention_tcgen05 != nullptr),
               "runner_bind: a module's entries come together");
    JK_REQUIRE((f.layernorm != nullptr) == (f.cast_rows != nullptr) && (f.layernorm != nullptr) == (f.glu != nullptr) &&
               (f.layernorm != nullptr) == (f.conv_qkv != nullptr) && (f.layernorm != nullptr) == (f.linear_scan != nullptr) &&
               (f.layernorm != nullptr) == (f.norm_gate != nullptr) && (f.layernorm != nullptr) == (f.err_mixers != nullptr) &&
               (f.layernorm != nullptr) == (f.token_shift != nullptr) && (f.layernorm != nullptr) == (f.act_rows != nullptr),
               "runner_bind: a module's entries come together");
    {
        void *const *first = (void *const *)&f.norm_add, *const *last = (void *const *)&f.err_blocks;
        for (void *const *e = first; e <= last; ++e)
            JK_REQUIRE((*e != nullptr) == (*first != nullptr), "runner_bind: a module's entries come together");
    }
    g_bound = true;
    return JK_OK;
}

static int g_launches = 0;      // kernels launched by the last jk_runner_run (the library's count as one each)
JK_EXPORT int jk_runner_launches() { return g_launches; }

#define RUN(module, call)                                                                                   \
    do {                                                                                                    \
        ++g_launches;                                                                                       \
        if (int rc_ = (call)) {                                                                             \
            snprintf(jk_error_buffer(), 512, "%s", g_fns.err_##module());                                   \
            return rc_;                                                                                     \
        }                                                                                                   \
    } while (0)

// ---- the library product: out[M, N] (float32) = act[M, K] * w[N, K]^T, bfloat16 operands --------------------
// cublasGemmEx with the library's own choice of kernel (it splits K for narrow outputs by itself), float32
// accumulation; the handle works in the caller's workspace so that nothing is allocated inside a capture.
static cublasHandle_t g_blas = nullptr;
static std::mutex g_blas_mutex;

static int lt_product(const void *act, const void *w, float *out, int M, int N, int K, const RunnerBuffers &b, cudaStream_t stream, int ldc = 0) {
    if (ldc <= 0) ldc = N;
    std::lock_guard<std::mutex> lock(g_blas_mutex);
    if (!g_blas && cublasCreate(&g_blas) != CUBLAS_STATUS_SUCCESS) JK_FAIL(JK_CUDA_ERROR, "runner: cublasCreate failed");
    JK_REQUIRE(b.workspace != nullptr && b.workspace_bytes > 0, "runner: the library's product needs a workspace");
    if (cublasSetStream(g_blas, stream) != CUBLAS_STATUS_SUCCESS ||
        cublasSetWorkspace(g_blas, b.workspace, (size_t)b.workspace_bytes) != CUBLAS_STATUS_SUCCESS)
        JK_FAIL(JK_CUDA_ERROR, "runner: the library refused the stream or the workspace");
    // row-major out[M, N] is column-major [N, M] = W^T (op T on the column-major [K, N]) * act (column-major [K, M])
    const float one = 1.f, zero = 0.f;
    ++g_launches;
    const cublasStatus_t st = cublasGemmEx(g_blas, CUBLAS_OP_T, CUBLAS_OP_N, N, M, K, &one, w, CUDA_R_16BF, K, act, CUDA_R_16BF, K,
                                           &zero, out, CUDA_R_32F, ldc, CUBLAS_COMPUTE_32F, CUBLAS_GEMM_DEFAULT_TENSOR_OP);
    if (st != CUBLAS_STATUS_SUCCESS) JK_FAIL(JK_CUDA_ERROR, "runner: the library's product of %d x %d x %d failed with %d", M, N, K, (int)st);
    return JK_OK;
}

namespace {

struct Run {
    const RunnerEnv &env;
    const RunnerStep &st;
    const RunnerBuffers &buf;
    cudaStream_t stream;
    bool pending = false;         // SLOT_DELTA holds a product that has not been added to the stream yet
    float pending_scale = 1.f;

    int elem() const { return env.dtype == JK_F32 ? 4 : 2; }
    bool tcgen05_bound() const { return g_fns.gemm_tcgen05 != nullptr; }
    jk::Route route(int rows, int n, int k, int kind) const {
        return jk::product_route(env.routing, rows, n, k, kind, g_fns.linear_small_supports(rows, n, k) != 0, tcgen05_bound());
    }
    // the slot's address, after a check that it holds `need` bytes
    int slot(int which, long long need, void **out, const char *what) const {
        JK_REQUIRE(which >= 0 && which < RUNNER_SLOTS && buf.slot[which] != nullptr, "runner: %s: slot %d is not there", what, which);
        JK_REQUIRE(need <= buf.bytes[which], "runner: %s needs %lld bytes in slot %d, which holds %lld", what, need, which, buf.bytes[which]);
        *out = buf.slot[which];
        return JK_OK;
    }
    float *x() const { return (float *)buf.slot[SLOT_X]; }
    float *delta() const { return (float *)buf.slot[SLOT_DELTA]; }
};

// out (float32 [rows, n]) = act * w^T (+ bias) by whichever kernel takes `rows`
// (`ldc` > 0: rows of out are that many floats apart)
int product_f32(Run &r, const void *act, const void *w, const float *bias, float *out, int rows, int n, int k, int ldc = 0) {
    if (ldc <= 0) ldc = n;
    if (r.env.dtype == JK_F32) {
        RUN(elementwise, g_fns.gemm_f32((const float *)act, k, (const float *)w, k, bias, out, ldc, rows, n, k, r.stream));
        return JK_OK;
    }
    // a bias outside q/k/v (whose bias the rotary kernel adds) does not occur in this architecture; no kernel adds one
    JK_REQUIRE(bias == nullptr, "runner: a bfloat16 product with a bias outside q/k/v is not built");
    const jk::Routing &ro = r.env.routing;
    switch (r.route(rows, n, k, jk::PRODUCT_F32)) {
        case jk::ROUTE_SMALL:
            RUN(linear_small, g_fns.linear_small(act, w, out, rows, n, k, ldc, 0, ro.sms, r.stream));
            break;
        case jk::ROUTE_SKINNY:
            RUN(gemm_tcgen05, g_fns.gemm_skinny(act, w, out, rows, n, k, ldc, 0, 1.f, r.env.status, ro.sms, r.stream));
            break;
        case jk::ROUTE_TCGEN05:
            RUN(gemm_tcgen05, g_fns.gemm_tcgen05(act, w, out, rows, n, k, ldc, 0, 1.f, r.env.status, ro.sms, r.stream));
            break;
        default:
            if (int rc = lt_product(act, w, out, rows, n, k, r.buf, r.stream, ldc)) return rc;
    }
    return JK_OK;
}

int flush_pending(Run &r, int T, int hidden) {
    if (!r.pending) return JK_OK;
    RUN(elementwise, g_fns.residual_add(r.x(), r.delta(), JK_F32, r.pending_scale, (long long)T * hidden, r.stream));
    r.pending = false;
    return JK_OK;
}

// Steps of few rows without norm kernels: three records in a row -- a product that adds into the stream, a norm over
// every row with factor 1, and a gate/up or q/k/v product that reads the norm's output -- run as two kernels.  The first
// adds itself into the float32 stream, writes bfloat16(x * norm weight) as the next product's activations and its
// tile's share of sum(x^2) per row into counters; the second multiplies its rows by 1 / sqrt(sum / width + eps) before
// its own epilogue.  The sums and the scaling are float32; what changes against the norm kernel is where the activations
// are rounded to bfloat16 (before the 1 / rms instead of after).
struct FusedNorm {
    const RunnerOp *norm = nullptr;       // the norm that the last residual product took over
    unsigned long long *sumsq = nullptr;
};

bool small_residual_ok(const Run &r, const RunnerOp &op, int T) {
    return r.env.dtype == JK_BF16 && r.env.fused_norms && T <= 16 && r.buf.sumsq != nullptr && op.out_slot == SLOT_X &&
           r.route(T, op.n, op.k, jk::PRODUCT_RESIDUAL) == jk::ROUTE_SMALL && g_fns.linear_small_norm_supports(T, op.n, op.k);
}
bool qkv_fusable(const Run &r, const RunnerOp &op) {
    return r.env.dtype == JK_BF16 && op.vec == nullptr && op.writes_cache && !op.interleaved && !r.env.routing.library_only;
}
bool consumer_takes_norm(const Run &r, const RunnerOp &norm, const RunnerOp &next, int T) {
    if (next.in_slot != norm.out_slot) return false;
    if (next.kind == OP_GATE_UP)
        return next.act != RUNNER_ACT_SWISH_CLAMP && r.route(T, next.n, next.k, jk::PRODUCT_SWIGLU) == jk::ROUTE_SMALL && g_fns.linear_small_norm_supports(T, next.n, next.k);
    if (next.kind == OP_QKV) return qkv_fusable(r, next) && g_fns.linear_small_qkv_supports(T, next.k, next.head_dim);
    return false;
}

int run_embed(Run &r, const RunnerOp &op) {
    void *out;
    if (int rc = r.slot(op.out_slot, 4LL * r.st.ntok * op.n, &out, "the embedding")) return rc;
    RUN(elementwise, g_fns.embed(r.st.tokens, r.st.ntok, op.w, op.w_dtype, op.n, op.scale, (float *)out, r.stream));
    return JK_OK;
}

int run_norm(Run &r, const RunnerOp &op) {
    const int rows = op.wanted_rows ? r.st.n_want : r.st.ntok;
    if (rows == 0) return JK_OK;
    void *out;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * rows * op.n, &out, "a norm")) return rc;
    // the pending product is added by the same kernel: into the stream when every row is normalised; a norm over the
    // wanted rows only reads stream + product for its rows and leaves both as they are
    RUN(elementwise, g_fns.add_rmsnorm(r.x(), r.pending ? r.delta() : nullptr, JK_F32, r.pending_scale, op.vec, op.eps, op.scale, out,
                                       r.env.dtype, op.wanted_rows ? r.st.want_rows : nullptr, rows, op.n, r.stream));
    if (!op.wanted_rows) r.pending = false;
    return JK_OK;
}

int run_qkv(Run &r, const RunnerOp &op, const FusedNorm &fused) {
    const int T = r.st.ntok, nq = op.n, d = op.k, nh = op.heads, nkvh = op.kv_heads, dh = op.head_dim;
    const jk::Routing &ro = r.env.routing;
    void *h, *q;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * T * d, &h, "q/k/v's activations")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * nh * dh, &q, "the queries")) return rc;
    const int *table = r.st.block_tables[op.cache_group];
    JK_REQUIRE(table != nullptr || !op.writes_cache, "runner: q/k/v writes the cache of group %d, whose block table the step lacks", op.cache_group);
    if (fused.norm != nullptr) {
        RUN(linear_small, g_fns.linear_small_qkv_norm(h, op.w, T, d, q, op.k_pages, op.v_pages, op.cos_table, op.sin_table,
                                                      r.st.positions, r.st.row_req, table, r.env.max_blocks, r.env.page_size, nh, nkvh,
                                                      dh, fused.sumsq, fused.norm->eps, ro.sms, r.stream));
        return JK_OK;
    }
    if (qkv_fusable(r, op)) {
        // the product's epilogue rotates and writes q and the cache itself: no float32 copy of the product, no rotary kernel
        if (r.tcgen05_bound() && jk::takes_tcgen05(ro, T, nq, d) && (dh == 64 || dh == 128)) {
            RUN(gemm_tcgen05, g_fns.gemm_tcgen05_qkv(h, op.w, T, d, q, op.k_pages, op.v_pages, op.cos_table, op.sin_table, r.st.positions,
                                                     r.st.row_req, table, r.env.max_blocks, r.env.page_size, nh, nkvh, dh,
                                                     r.env.status, ro.sms, r.stream));
            return JK_OK;
        }
        if (T <= 16 && g_fns.linear_small_qkv_supports(T, d, dh)) {
            RUN(linear_small, g_fns.linear_small_qkv(h, op.w, T, d, q, op.k_pages, op.v_pages, op.cos_table, op.sin_table, r.st.positions,
                                                     r.st.row_req, table, r.env.max_blocks, r.env.page_size, nh, nkvh, dh, ro.sms,
                                                     r.stream));
            return JK_OK;
        }
    }
    void *tmp;
    if (int rc = r.slot(SLOT_TMP, 4LL * T * nq, &tmp, "the q/k/v product")) return rc;
    if (int rc = product_f32(r, h, op.w, nullptr, (float *)tmp, T, nq, d)) return rc;
    RUN(elementwise, g_fns.rope_kv(tmp, JK_F32, nq, op.vec, r.st.positions, r.st.row_req, table, r.env.max_blocks, r.env.page_size,
                                   op.cos_table, op.sin_table, op.interleaved, q, op.k_pages, op.v_pages, r.env.dtype, T, nh, nkvh, dh,
                                   op.writes_cache, r.stream));
    return JK_OK;
}

int run_attention(Run &r, const RunnerOp &op) {
    const int T = r.st.ntok, nh = op.heads, nkvh = op.kv_heads, dh = op.head_dim, page = r.env.page_size;
    const int dv = op.v_head_dim > 0 ? op.v_head_dim : dh;
    void *q, *o;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * T * nh * dh, &q, "the queries")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * nh * dv, &o, "attention's output")) return rc;
    const float *gate = nullptr;
    if (op.gated) {
        void *u;
        if (int rc = r.slot(SLOT_TMP, 4LL * T * op.ld, &u, "the projection that holds attention's gate")) return rc;
        gate = (const float *)u + op.g_off;
    }
    const int *table = r.st.block_tables[op.cache_group];
    JK_REQUIRE(table != nullptr, "runner: attention reads the cache of group %d, whose block table the step lacks", op.cache_group);
    const int n_short = r.st.list_n[op.list_short], n_tiles = r.st.list_n[op.list_tiles];
    const int *short_rows = r.st.lists[op.list_short], *tiles = r.st.lists[op.list_tiles];
    const bool tc = !r.env.legacy_tensor_cores && g_fns.attention_tcgen05 != nullptr && jk::attention_tcgen05_takes(dh, page, dv);
    bool fast = r.env.dtype == JK_BF16 && !r.env.plain_attention && (n_short > 0 || n_tiles > 0) && dh % 8 == 0 && dh <= 256;
    // values of another size than the keys: the tcgen05 tiles and the split decode on tensor cores take them (padded to 64 or
    // 128), the mma.sync tiles do not; else the row kernel (a sink, a gate, capped scores and kept first keys every kernel takes)
    if (dv != dh && !jk::attention_unlike_heads(dh, dv)) fast = false;
    if (fast && n_tiles > 0 && !(tc || (dv == dh && g_fns.attention_prefill_supports(dh)))) fast = false;
    if (!fast) {
        // one warp per (row, head): float32, and every shape the tensor-core kernels are not built for
        RUN(attention, g_fns.attention_rows(q, op.k_pages, op.v_pages, o, r.env.dtype, r.st.positions, r.st.row_req, table,
                                            r.env.max_blocks, page, T, nh, nkvh, dh, op.softmax_scale, op.window, dv, op.sink, gate, op.ld,
                                            op.cap, op.keep_first, op.sink_w, op.gated == 2, r.stream));
        return JK_OK;
    }
    if (n_tiles > 0) {
        if (tc)
            RUN(attention_tcgen05, g_fns.attention_tcgen05(q, op.k_pages, op.v_pages, o, tiles, n_tiles, T, r.st.req_start, r.st.req_pos,
                                                           table, r.env.max_blocks, op.num_pages, page, nh, nkvh, dh, op.softmax_scale,
                                                           op.window, r.env.status, op.sink, gate, op.ld, op.cap, op.keep_first, op.sink_w,
                                                           op.gated == 2, dv, r.stream));
        else
            RUN(attention, g_fns.attention_prefill(q, op.k_pages, op.v_pages, o, tiles, n_tiles, jk::TILE_ROWS, r.st.req_start,
                                                   r.st.req_pos, table, r.env.max_blocks, page, nh, nkvh, dh, op.softmax_scale,
                                                   op.window, op.sink, gate, op.ld, op.cap, op.keep_first, op.sink_w, op.gated == 2, r.stream));
    }
    if (n_short > 0) {
        const int context = r.st.context > 0 ? r.st.context : op.max_positions;
        const int splits = jk::decode_splits(n_short, nkvh, nh / nkvh, jk::decode_keys_hint(context, std::abs(op.window)), r.env.routing.sms, jk::decode_head(dh, dv));
        void *scratch = nullptr;
        const long long need = 4 * jk::decode_scratch_floats(n_short, nh, dv, splits);
        if (need > 0)
            if (int rc = r.slot(SLOT_DECODE, need, &scratch, "the split-key attention's partial results")) return rc;
        RUN(attention, g_fns.attention_decode(q, op.k_pages, op.v_pages, o, (float *)scratch, short_rows, n_short, r.st.positions,
                                              r.st.row_req, table, r.env.max_blocks, page, nh, nkvh, dh, op.softmax_scale, op.window,
                                              splits, op.sink, gate, op.ld, op.cap, op.keep_first, op.sink_w, op.gated == 2, dv, r.stream));
    }
    return JK_OK;
}

// stream += scale * (in w^T): in the product's epilogue where that exists, else left pending for the next norm
int run_residual(Run &r, const RunnerOp &op, const RunnerOp *norm, const RunnerOp *consumer, int op_index, FusedNorm *fused) {
    const int T = r.st.ntok;
    const jk::Routing &ro = r.env.routing;
    void *act;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * T * op.k, &act, "a product's activations")) return rc;
    JK_REQUIRE(op.out_slot == SLOT_X, "runner: a residual product adds into the stream");
    if (int rc = flush_pending(r, T, op.n)) return rc;
    if (small_residual_ok(r, op, T)) {
        const bool take_norm = norm != nullptr && norm->kind == OP_NORM && !norm->wanted_rows && norm->scale == 1.f && norm->n == op.n &&
                               consumer != nullptr && consumer_takes_norm(r, *norm, *consumer, T) && op_index < r.buf.sumsq_rows;
        void *h = nullptr;
        unsigned long long *ss = nullptr;
        if (take_norm) {
            if (int rc = r.slot(norm->out_slot, 2LL * T * op.n, &h, "a norm")) return rc;
            ss = r.buf.sumsq + (size_t)op_index * 16;
            fused->norm = norm;
            fused->sumsq = ss;
        }
        RUN(linear_small, g_fns.linear_small_norm(act, op.w, r.x(), T, op.n, op.k, op.n, 3, nullptr, 0.f, h, take_norm ? norm->vec : nullptr,
                                                  ss, op.scale, r.env.status, ro.sms, r.stream));
        return JK_OK;
    }
    if (r.env.dtype == JK_BF16) {
        const jk::Route route = r.route(T, op.n, op.k, jk::PRODUCT_RESIDUAL);
        if (route == jk::ROUTE_SKINNY) {
            RUN(gemm_tcgen05, g_fns.gemm_skinny(act, op.w, r.x(), T, op.n, op.k, op.n, 2, op.scale, r.env.status, ro.sms, r.stream));
            return JK_OK;
        }
        if (route == jk::ROUTE_TCGEN05) {
            RUN(gemm_tcgen05, g_fns.gemm_tcgen05(act, op.w, r.x(), T, op.n, op.k, op.n, 2, op.scale, r.env.status, ro.sms, r.stream));
            return JK_OK;
        }
    }
    void *delta;
    if (int rc = r.slot(SLOT_DELTA, 4LL * T * op.n, &delta, "a product that waits for the next norm")) return rc;
    if (int rc = product_f32(r, act, op.w, nullptr, (float *)delta, T, op.n, op.k)) return rc;
    r.pending = true;
    r.pending_scale = op.scale;
    return JK_OK;
}

int run_gate_up(Run &r, const RunnerOp &op, const FusedNorm &fused) {
    const int T = r.st.ntok, di = op.n, d = op.k;
    const jk::Routing &ro = r.env.routing;
    void *h, *act;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * T * d, &h, "gate/up's activations")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * di, &act, "the feed-forward's inner activations")) return rc;
    // the gate's activation rides above the epilogue's code (common.cuh: gated_unit)
    JK_REQUIRE(op.act == RUNNER_ACT_NONE || op.act == RUNNER_ACT_SILU || op.act == RUNNER_ACT_GELU_TANH || op.act == RUNNER_ACT_RELU ||
               op.act == RUNNER_ACT_SWISH_CLAMP, "runner: a gated unit with activation %d is not built", op.act);
    const bool clamped = op.act == RUNNER_ACT_SWISH_CLAMP;      // no product has this unit in its epilogue: product, then the unit's kernel
    const bool other_gate = op.act == RUNNER_ACT_GELU_TANH || op.act == RUNNER_ACT_RELU || clamped;      // not silu: the unfused unit is the mixers module's
    const int gate_bits = other_gate ? (op.act << 8) : 0;
    if (fused.norm != nullptr && !clamped) {
        RUN(linear_small, g_fns.linear_small_norm(h, op.w, act, T, di, d, di, 1 | gate_bits, fused.sumsq, fused.norm->eps, nullptr, nullptr, nullptr,
                                                  1.f, r.env.status, ro.sms, r.stream));
        return JK_OK;
    }
    if (r.env.dtype == JK_BF16 && !clamped) {
        switch (r.route(T, di, d, jk::PRODUCT_SWIGLU)) {
            case jk::ROUTE_SMALL:
                RUN(linear_small, g_fns.linear_small(h, op.w, act, T, di, d, di, 1 | gate_bits, ro.sms, r.stream));
                return JK_OK;
            case jk::ROUTE_SKINNY:
                RUN(gemm_tcgen05, g_fns.gemm_skinny(h, op.w, act, T, di, d, di, 3 | gate_bits, 1.f, r.env.status, ro.sms, r.stream));
                return JK_OK;
            case jk::ROUTE_TCGEN05:
                RUN(gemm_tcgen05, g_fns.gemm_tcgen05(h, op.w, act, T, di, d, di, 3 | gate_bits, 1.f, r.env.status, ro.sms, r.stream));
                return JK_OK;
            default:
                break;
        }
    }
    void *tmp;
    if (int rc = r.slot(SLOT_TMP, 4LL * T * 2 * di, &tmp, "the gate/up product")) return rc;
    if (r.env.dtype == JK_F32) {
        RUN(elementwise, g_fns.gemm_f32((const float *)h, d, (const float *)op.w, d, nullptr, (float *)tmp, 2 * di, T, 2 * di, d, r.stream));
    } else if (clamped) {
        if (int rc = product_f32(r, h, op.w, nullptr, (float *)tmp, T, 2 * di, d)) return rc;       // by the rows' route, float32 sums
    } else {
        if (int rc = lt_product(h, op.w, (float *)tmp, T, 2 * di, d, r.buf, r.stream)) return rc;
    }
    if (other_gate) {
        JK_REQUIRE(g_fns.glu != nullptr, "runner: the unfused gated unit with activation %d needs the mixers module", op.act);
        RUN(mixers, g_fns.glu((const float *)tmp, act, r.env.dtype, T, di, op.act, op.limit, r.stream));
        return JK_OK;
    }
    RUN(elementwise, g_fns.swiglu(tmp, JK_F32, act, r.env.dtype, T, di, r.stream));
    return JK_OK;
}

int run_linear(Run &r, const RunnerOp &op) {
    const int rows = op.wanted_rows ? r.st.n_want : r.st.ntok;
    if (rows == 0) return JK_OK;
    void *in, *out;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * rows * op.k * (op.in_part + 1), &in, "a product's activations")) return rc;
    if (op.out_slot == SLOT_DELTA && !op.wanted_rows)       // a product that waits there goes into the stream first
        if (int rc = flush_pending(r, rows, op.n)) return rc;
    in = (char *)in + (size_t)r.elem() * rows * op.k * op.in_part;
    if (op.ld > 0) {        // a column range of wider rows
        JK_REQUIRE(op.out_off >= 0 && op.out_off + op.n <= op.ld, "runner: a product writes columns %d .. %d of rows of %d", op.out_off, op.out_off + op.n, op.ld);
        if (int rc = r.slot(op.out_slot, 4LL * rows * op.ld, &out, "a product's output")) return rc;
        return product_f32(r, in, op.w, op.vec, (float *)out + op.out_off, rows, op.n, op.k, op.ld);
    }
    if (int rc = r.slot(op.out_slot, 4LL * rows * op.n, &out, "a product's output")) return rc;
    return product_f32(r, in, op.w, op.vec, (float *)out, rows, op.n, op.k);
}

// Steps of few rows: products in a row that read neighbouring parts of one slot (a mixer whose projections each read their
// own mixture of its input), with neighbouring rows of one weight matrix, into neighbouring column ranges of the same
// float32 rows, run as one launch of the few-row kernel.  Returns how many records from ops[i] on it ran (0: none; the
// caller runs them one by one).
int run_linears_together(Run &r, const RunnerOp *ops, int i, int end, int *ran) {
    *ran = 0;
    const RunnerOp &op = ops[i];
    const int rows = r.st.ntok;
    if (g_fns.linear_small_parts == nullptr || g_fns.linear_small_parts_supports == nullptr || r.env.dtype != JK_BF16 || rows > 16 || rows == 0 ||
        op.wanted_rows || op.ld <= 0 || op.in_part != 0 || op.vec != nullptr)
        return JK_OK;
    int ends[8], n = 0, width = 0;
    for (int j = i; j < end && n < 8; ++j) {
        const RunnerOp &o = ops[j];
        if (o.kind != OP_LINEAR || o.wanted_rows || o.vec != nullptr || o.in_slot != op.in_slot || o.out_slot != op.out_slot || o.ld != op.ld ||
            o.k != op.k || o.in_part != n || o.out_off != op.out_off + width ||
            (const char *)o.w != (const char *)op.w + (size_t)width * op.k * r.elem())
            break;
        if (n > 0 && width % 16 != 0) break;        // a tile of 16 features lies in one part
        width += o.n;
        ends[n++] = width;
    }
    if (n < 2) return JK_OK;
    while (n >= 2 && r.route(rows, width, op.k, jk::PRODUCT_F32) != jk::ROUTE_SMALL) width = ends[--n - 1];
    if (n < 2 || !g_fns.linear_small_parts_supports(rows, width, op.k)) return JK_OK;
    void *in, *out;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * rows * op.k * n, &in, "the products' activations")) return rc;
    if (int rc = r.slot(op.out_slot, 4LL * rows * op.ld, &out, "the products' output")) return rc;
    JK_REQUIRE(op.out_off >= 0 && op.out_off + width <= op.ld, "runner: products write columns %d .. %d of rows of %d", op.out_off, op.out_off + width, op.ld);
    RUN(linear_small, g_fns.linear_small_parts(in, (long long)rows * op.k, ends, n, op.w, (float *)out + op.out_off, rows, width, op.k, op.ld,
                                               r.env.routing.sms, r.stream));
    *ran = n;
    return JK_OK;
}

// ---- records of csrc/mixers.cu -------------------------------------------------------------------------------
int need_mixers(const char *what) {
    JK_REQUIRE(g_fns.layernorm != nullptr, "runner: %s needs the mixers module, which was not bound", what);
    return JK_OK;
}

int run_cast(Run &r, const RunnerOp &op) {
    if (int rc = need_mixers("a cast of the stream")) return rc;
    const int T = r.st.ntok;
    void *out;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n, &out, "the stream as activations")) return rc;
    if (int rc = flush_pending(r, T, op.n)) return rc;
    RUN(mixers, g_fns.cast_rows(r.x(), out, r.env.dtype, (long long)T * op.n, r.stream));
    return JK_OK;
}

int run_layernorm(Run &r, const RunnerOp &op) {
    if (int rc = need_mixers("a layer norm")) return rc;
    const int T = r.st.ntok;
    if (op.in_slot == SLOT_DELTA) {         // the norm of a sublayer's output, added into the stream
        void *delta, *h = nullptr;
        if (int rc = r.slot(SLOT_DELTA, 4LL * T * op.n, &delta, "a sublayer's output")) return rc;
        if (op.out_slot >= 0)
            if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n, &h, "the stream as activations")) return rc;
        JK_REQUIRE(!r.pending, "runner: a layer norm over a sublayer's output while another product waits to be added");
        RUN(mixers, g_fns.layernorm((const float *)delta, nullptr, T, op.n, op.vec, op.bias, op.eps, r.x(), h, r.env.dtype, r.stream));
        return JK_OK;
    }
    const int rows = op.wanted_rows ? r.st.n_want : T;
    if (rows == 0) return JK_OK;
    void *out;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * rows * op.n, &out, "a norm")) return rc;
    if (int rc = flush_pending(r, T, op.n)) return rc;
    RUN(mixers, g_fns.layernorm(r.x(), op.wanted_rows ? r.st.want_rows : nullptr, rows, op.n, op.vec, op.bias, op.eps, nullptr, out,
                                r.env.dtype, r.stream));
    return JK_OK;
}

int run_conv_qkv(Run &r, const RunnerOp &op) {
    if (int rc = need_mixers("a convolved q/k/v")) return rc;
    const int T = r.st.ntok, dv = op.v_head_dim > 0 ? op.v_head_dim : op.head_dim;
    void *u, *q;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.ld, &u, "the q/k/v projection")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.heads * op.head_dim, &q, "the queries")) return rc;
    const int *table = op.has_kv ? r.st.block_tables[op.cache_group] : nullptr;
    JK_REQUIRE(!op.has_kv || table != nullptr, "runner: q/k/v writes the cache of group %d, whose block table the step lacks", op.cache_group);
    JK_REQUIRE(r.st.slot_ids != nullptr || op.state == nullptr, "runner: a convolution keeps tails, but the step names no state slots");
    RUN(mixers, g_fns.conv_qkv((const float *)u, op.ld, op.q_off, op.k_off, op.v_off, op.heads, op.kv_heads, op.head_dim, dv, op.has_kv,
                               op.conv_q, op.conv_k, op.conv_v, op.taps, op.norm_q, op.norm_k, op.eps, op.freq, op.rot_dims, op.state,
                               r.st.positions, r.st.row_req, r.st.req_start, r.st.slot_ids, table, r.env.max_blocks, r.env.page_size, q,
                               op.k_pages, op.v_pages, r.env.dtype, T, r.st.nreq, op.rot_half, op.rot_mag, op.head_norm, op.bias, op.temp, r.stream));
    if (op.taps > 1 && T > r.st.nreq) ++g_launches;      // the tails' kernel
    return JK_OK;
}

int run_linear_attention(Run &r, const RunnerOp &op) {
    if (int rc = need_mixers("a linear attention")) return rc;
    const int T = r.st.ntok, dv = op.v_head_dim > 0 ? op.v_head_dim : op.head_dim;
    void *u, *mix, *out;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.ld, &u, "the q/k/v projection")) return rc;
    if (int rc = r.slot(SLOT_MIX, 4LL * T * op.heads * dv, &mix, "a recurrence's output")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.heads * dv, &out, "a linear attention's output")) return rc;
    JK_REQUIRE(r.st.slot_ids != nullptr && op.state != nullptr, "runner: a recurrence without its state slots");
    const int n_pieces = r.st.list_n[op.list_tiles];
    void *scratch = nullptr;
    long long scratch_floats = 0;
    if (n_pieces > 0) {
        scratch_floats = (long long)n_pieces * op.heads * op.head_dim * dv + (op.rank ? (long long)T * op.heads * op.head_dim : 0);
        if (int rc = r.slot(SLOT_SCAN, 4 * scratch_floats, &scratch, "the pieces of a recurrence")) return rc;
    }
    RUN(mixers, g_fns.linear_scan((const float *)u, op.ld, op.q_off, op.k_off, op.v_off, op.heads, op.head_dim, dv, op.act, op.q_scale,
                                  op.decay, op.w2, r.env.dtype, op.b2, op.r_off, op.rank, op.tau, op.state, r.st.req_start, r.st.slot_ids,
                                  r.st.nreq, T, (float *)mix, r.st.lists[op.list_short], r.st.list_n[op.list_short],
                                  r.st.lists[op.list_tiles], n_pieces, r.st.lists[op.list_aux], r.st.list_n[op.list_aux],
                                  (float *)scratch, scratch_floats, r.env.routing.sms, op.bonus, op.decay_form, op.rank_act, r.stream));
    // the carry and the prefix kernels; pieces that run as tiled products have a kernel beside the one of the requests that run in one go
    if (n_pieces > 0)
        g_launches += 2 + (r.st.list_n[op.list_short] > 0 && jk::scan_runs_tiled(op.head_dim, dv, op.ld, op.q_off, op.k_off, op.v_off, op.w2 != nullptr, op.bonus != nullptr) ? 1 : 0);
    RUN(mixers, g_fns.norm_gate((const float *)mix, (const float *)u, op.ld, op.g_off, op.vec, op.eps, op.heads, dv, op.per_head_norm,
                                op.gate_act, out, r.env.dtype, T, r.stream));
    return JK_OK;
}

// ---- records of csrc/blocks.cu --------------------------------------------------------------------------------
int need_blocks(const char *what) {
    JK_REQUIRE(g_fns.norm_add != nullptr, "runner: %s needs the blocks module, which was not bound", what);
    return JK_OK;
}

int run_norm_add(Run &r, const RunnerOp &op) {
    if (int rc = need_blocks("a norm that adds a sublayer's output")) return rc;
    const int T = r.st.ntok;
    void *delta, *h = nullptr;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.n, &delta, "a sublayer's output")) return rc;
    if (op.out_slot >= 0)
        if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n, &h, "the next sublayer's input")) return rc;
    JK_REQUIRE(!r.pending, "runner: a norm over a sublayer's output while another product waits to be added");
    void *h2 = nullptr;
    if (op.out2_slot >= 0)
        if (int rc = r.slot(op.out2_slot, (long long)r.elem() * T * op.n, &h2, "the input of the sublayer beside the next")) return rc;
    RUN(blocks, g_fns.norm_add((const float *)delta, r.x(), op.vec, op.eps, op.vec2, op.eps2, h, op.vec3, h2, r.env.dtype, T, op.n, r.stream));
    return JK_OK;
}

int run_reinject(Run &r, const RunnerOp &op) {
    if (int rc = need_blocks("feeding the embedding in again")) return rc;
    const int T = r.st.ntok;
    void *x0, *both;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.n, &x0, "the embedding's output")) return rc;
    if (int rc = r.slot(SLOT_ACT, (long long)r.elem() * T * op.k, &both, "the stream beside the embedding's output")) return rc;
    JK_REQUIRE(op.k == 2 * op.n, "runner: feeding the embedding in again takes a matrix of %d x %d, found %d x %d", op.n, 2 * op.n, op.n, op.k);
    if (int rc = flush_pending(r, T, op.n)) return rc;
    RUN(blocks, g_fns.concat_cast(r.x(), (const float *)x0, both, r.env.dtype, T, op.n, r.stream));
    if (r.env.dtype == JK_F32) {
        RUN(elementwise, g_fns.gemm_f32((const float *)both, op.k, (const float *)op.w, op.k, op.vec, r.x(), op.n, T, op.n, op.k, r.stream));
        return JK_OK;
    }
    if (int rc = product_f32(r, both, op.w, nullptr, r.x(), T, op.n, op.k)) return rc;
    if (op.vec != nullptr) RUN(blocks, g_fns.add_bias_rows(r.x(), op.vec, T, op.n, r.stream));
    return JK_OK;
}

int run_latent_qkv(Run &r, const RunnerOp &op) {
    if (int rc = need_blocks("a latent attention's queries")) return rc;
    const int T = r.st.ntok, H = op.heads, D = op.rank + op.rot_width;
    void *u, *q_full, *q_plain;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.ld, &u, "the query and latent projection")) return rc;
    const bool queries_only = op.k_off < 0;
    if (op.q_rank > 0) {        // the queries' own latent vector, normed; the heads' queries are made by the records that follow
        q_full = nullptr;
        if (int rc = r.slot(op.out2_slot, (long long)r.elem() * T * op.q_rank, &q_plain, "the queries' latent vector")) return rc;
    } else {
        if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * H * D, &q_full, "the queries")) return rc;
        if (int rc = r.slot(op.out2_slot, (long long)r.elem() * T * H * op.head_dim, &q_plain, "the queries' plain parts")) return rc;
    }
    const int *table = queries_only ? nullptr : r.st.block_tables[op.cache_group];
    JK_REQUIRE(table != nullptr || queries_only, "runner: a latent attention writes the cache of group %d, whose block table the step lacks", op.cache_group);
    RUN(blocks, g_fns.latent_qkv((const float *)u, op.ld, op.q_off, op.k_off, H, op.head_dim, op.rot_width, op.rank, op.rot_dims, op.freq,
                                 op.rot_mag, op.norm_k, op.eps, r.st.positions, r.st.row_req, table, r.env.max_blocks, r.env.page_size,
                                 q_plain, q_full, op.k_pages, r.env.dtype, T, op.q_rank > 0 ? op.norm_q : nullptr, op.q_rank, op.rot_half, r.stream));
    return JK_OK;
}

int run_head_linear(Run &r, const RunnerOp &op) {
    if (int rc = need_blocks("a product per head")) return rc;
    const int T = r.st.ntok;
    void *in, *out;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * T * op.heads * op.k, &in, "a per-head product's operand")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.heads * op.out_hs, &out, "a per-head product's output")) return rc;
    const float *gate = nullptr;
    if (op.gated) {
        void *u;
        if (int rc = r.slot(SLOT_TMP, 4LL * T * op.ld, &u, "the projection that holds the gate")) return rc;
        gate = (const float *)u + op.g_off;
    }
    RUN(blocks, g_fns.head_linear(in, op.w, out, r.env.dtype, T, op.heads, op.n, op.k, op.out_hs, gate, op.ld, op.gated == 2, r.stream));
    return JK_OK;
}

// How many ranges the keys of a row are cut into: steps of few rows fill the SMs with ranges of at least 256 keys (128
// where a window bounds a row's keys: a launch's time is that of one range, and a window leaves few ranges of 256).
int latent_splits(int T, int heads, int context, int sms, int least = 256) {
    if (T > 16) return 1;
    const int blocks = T * ((heads + 7) / 8);
    const int want = (2 * sms + blocks - 1) / blocks, by_length = (context + least - 1) / least;
    return std::max(1, std::min(std::min(want, by_length), 64));
}

int run_latent_attention(Run &r, const RunnerOp &op) {
    if (int rc = need_blocks("a latent attention")) return rc;
    const int T = r.st.ntok, H = op.heads, D = op.rank + op.rot_width;
    void *q, *o;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * T * H * D, &q, "the queries")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * H * op.rank, &o, "a latent attention's output")) return rc;
    const int *table = r.st.block_tables[op.cache_group];
    JK_REQUIRE(table != nullptr, "runner: a latent attention reads the cache of group %d, whose block table the step lacks", op.cache_group);
    int reach = r.st.context > 0 ? r.st.context : op.max_positions;
    if (op.window > 0) reach = std::min(reach, op.window);
    const int splits = latent_splits(T, H, reach, r.env.routing.sms, op.window > 0 ? 128 : 256);
    void *part = nullptr;
    if (splits > 1)
        if (int rc = r.slot(SLOT_DECODE, 4 * g_fns.latent_attention_scratch(T, H, op.rank, splits), &part, "the ranges of a latent attention")) return rc;
    RUN(blocks, g_fns.latent_attention(q, op.k_pages, o, (float *)part, r.env.dtype, r.st.positions, r.st.row_req, table, r.env.max_blocks,
                                       r.env.page_size, T, H, op.rank, op.rot_width, op.softmax_scale, splits, r.st.req_start, r.st.nreq, op.window, op.sink_w, r.stream));
    if (splits > 1) ++g_launches;
    return JK_OK;
}

int run_causal_conv(Run &r, const RunnerOp &op) {
    if (int rc = need_blocks("a convolution over time")) return rc;
    const int T = r.st.ntok;
    void *u, *y32 = nullptr, *yT = nullptr;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.ld, &u, "a convolution's input")) return rc;
    if (op.out2_slot >= 0)
        if (int rc = r.slot(op.out2_slot, 4LL * T * op.n, &y32, "a convolution's float32 output")) return rc;
    if (op.out_slot >= 0)
        if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n, &yT, "a convolution's output")) return rc;
    JK_REQUIRE(r.st.slot_ids != nullptr || op.taps <= 1, "runner: a convolution keeps tails, but the step names no state slots");
    RUN(blocks, g_fns.causal_conv((const float *)u, op.ld, op.q_off, op.n, op.conv_q, op.bias, op.taps, op.act, op.state, r.st.row_req,
                                  r.st.req_start, r.st.slot_ids, (float *)y32, yT, r.env.dtype, T, r.st.nreq, op.in_bias, r.stream));
    if (op.taps > 1 && T > r.st.nreq) ++g_launches;
    return JK_OK;
}

int run_selective_scan(Run &r, const RunnerOp &op) {
    if (int rc = need_blocks("a selective scan")) return rc;
    const int T = r.st.ntok, ld_low = op.rank + 2 * op.k;
    void *x, *low, *u, *out;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.n, &x, "a scan's input")) return rc;
    if (int rc = r.slot(op.in2_slot, 4LL * T * ld_low, &low, "a scan's step sizes and maps")) return rc;
    if (int rc = r.slot(SLOT_TMP, 4LL * T * op.ld, &u, "the projection that holds a scan's gate")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n, &out, "a scan's output")) return rc;
    JK_REQUIRE(r.st.slot_ids != nullptr && op.state != nullptr, "runner: a scan without its state slots");
    RUN(blocks, g_fns.selective_scan((const float *)x, (const float *)low, ld_low, op.rank, op.k, op.n, (const float *)u + op.g_off, op.ld,
                                     op.w2, op.b2, op.decay, op.vec, op.state, r.st.req_start, r.st.slot_ids, r.st.nreq, out,
                                     r.env.dtype, (float *)u + op.q_off, op.ld, T, r.stream));
    ++g_launches;       // the step sizes' product
    return JK_OK;
}

int run_experts(Run &r, const RunnerOp &op) {
    if (int rc = need_blocks("routed experts")) return rc;
    const int T = r.st.ntok;
    void *h, *delta, *route, *act, *y;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * T * op.n, &h, "the experts' input")) return rc;
    if (int rc = r.slot(SLOT_DELTA, 4LL * T * op.n, &delta, "the experts' output")) return rc;
    const bool adds = op.into_stream == 2;      // the sum goes into the stream by its own kernel, with a product that waits
    if (int rc = r.slot(SLOT_ROUTE, 4 * g_fns.routed_experts_workspace(T, op.experts + op.identity, op.top), &route, "the rows' choice of experts")) return rc;
    if (int rc = r.slot(SLOT_ACT, (long long)r.elem() * T * op.top * op.ff, &act, "the experts' inner activations")) return rc;
    if (int rc = r.slot(SLOT_TMP, 4LL * T * op.top * op.n, &y, "the experts' results")) return rc;
    JK_REQUIRE(!r.pending || (adds && !op.add), "runner: routed experts while another product waits to be added");
    RUN(blocks, g_fns.routed_experts(h, op.vec, op.w, op.w3, (float *)delta, op.add, r.env.dtype, T, op.n, op.ff, op.experts, op.top, op.act,
                                     (int *)route, act, (float *)y, op.score_form, op.limit, op.router_bias, op.gate_w, op.identity, op.group_count, op.group_keep,
                                   op.correction, adds ? r.x() : nullptr, op.scale, r.pending ? (const float *)delta : nullptr, r.pending_scale,
                                   op.score_scale > 0.f ? op.score_scale : 1.f, r.stream));
    g_launches += g_fns.routed_experts_launches() - 1;
    if (adds) {
        r.pending = false;
    } else if (op.into_stream) {       // a block without a norm on the sublayer's output: the next norm adds it
        r.pending = true;
        r.pending_scale = 1.f;
    }
    return JK_OK;
}

int run_norm_pair(Run &r, const RunnerOp &op) {
    JK_REQUIRE(g_fns.norm_pair != nullptr, "runner: a pair of norms needs the blocks module, which was not bound");
    const int T = r.st.ntok;
    void *h, *h2 = nullptr;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n, &h, "the first norm of a pair")) return rc;
    if (op.out2_slot >= 0)
        if (int rc = r.slot(op.out2_slot, (long long)r.elem() * T * op.n, &h2, "the second norm of a pair")) return rc;
    JK_REQUIRE(op.bias == nullptr || (op.state != nullptr && r.st.slot_ids != nullptr), "runner: a token shift without its state slots");
    if (int rc = flush_pending(r, T, op.n)) return rc;
    RUN(blocks, g_fns.norm_pair(r.x(), op.vec, op.bias, op.eps, op.vec2, op.eps2, op.state, r.st.row_req, r.st.req_start, r.st.req_pos, r.st.slot_ids,
                                h, h2, r.env.dtype, T, op.n, r.stream));
    return JK_OK;
}

int run_token_shift(Run &r, const RunnerOp &op) {
    if (int rc = need_mixers("a token shift")) return rc;
    const int T = r.st.ntok;
    void *h, *out;
    if (int rc = r.slot(op.in_slot, (long long)r.elem() * T * op.n, &h, "a token shift's input")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n * op.heads, &out, "the shifted mixtures")) return rc;
    JK_REQUIRE(r.st.slot_ids != nullptr && op.state != nullptr && op.vec != nullptr, "runner: a token shift without its state slots or mixing vectors");
    RUN(mixers, g_fns.token_shift(h, op.vec, op.state, r.st.row_req, r.st.req_start, r.st.slot_ids, out, r.env.dtype, T, r.st.nreq, op.n, op.heads,
                                  r.stream));
    ++g_launches;       // the kernel that moves the kept rows on
    return JK_OK;
}

int run_activate(Run &r, const RunnerOp &op) {
    if (int rc = need_mixers("an activation between two products")) return rc;
    const int T = r.st.ntok, ld = op.ld > 0 ? op.ld : op.n;
    void *u, *out;
    if (int rc = r.slot(op.in_slot, 4LL * T * ld, &u, "an activation's input")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n, &out, "an activation's output")) return rc;
    RUN(mixers, g_fns.act_rows((const float *)u, ld, out, r.env.dtype, T, op.n, op.act, op.w, op.k, op.g_off, r.st.tokens, r.stream));
    return JK_OK;
}

int run_add_rows(Run &r, const RunnerOp &op) {
    JK_REQUIRE(g_fns.add_rows != nullptr, "runner: rows of a table added to the stream need the blocks module, which was not bound");
    const int T = r.st.ntok;
    void *x;
    if (int rc = r.slot(SLOT_X, 4LL * T * op.n, &x, "the stream")) return rc;
    if (int rc = flush_pending(r, T, op.n)) return rc;
    RUN(blocks, g_fns.add_rows((float *)x, op.w, op.w_dtype, op.k, op.fixed_row < 0 ? r.st.positions : nullptr, op.fixed_row, T, op.n, r.stream));
    return JK_OK;
}

// DELTA_RULE: ld = width of the convolved rows in in_slot (q at q_off, k at k_off, v at v_off); r_off = width of SLOT_TMP's rows
// (the write strength's logit at b_off + h, the decay's at a_off + h, the gate at g_off)
int run_delta_rule(Run &r, const RunnerOp &op) {
    if (int rc = need_mixers("a delta rule")) return rc;
    JK_REQUIRE(g_fns.delta_rule != nullptr && g_fns.delta_rule_scratch != nullptr, "runner: a delta rule needs its kernel, which was not bound");
    const int T = r.st.ntok, dv = op.v_head_dim;
    void *c, *u, *mix, *out;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.ld, &c, "the convolved q/k/v")) return rc;
    if (int rc = r.slot(SLOT_TMP, 4LL * T * op.r_off, &u, "the projection that holds a delta rule's logits and gate")) return rc;
    // the slot of the recurrences' scratch holds the output before its norm, then what the rows' preparation leaves
    const long long o_floats = ((long long)T * op.heads * dv + 3) / 4 * 4;
    const long long prep_floats = g_fns.delta_rule_scratch(T, op.heads, op.groups, op.head_dim);
    if (int rc = r.slot(SLOT_SCAN, 4 * (o_floats + prep_floats), &mix, "a recurrence's output and its prepared rows")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.heads * dv, &out, "a delta rule's output")) return rc;
    JK_REQUIRE(r.st.slot_ids != nullptr && op.state != nullptr, "runner: a recurrence without its state slots");
    RUN(mixers, g_fns.delta_rule((const float *)c, op.ld, op.q_off, op.k_off, op.v_off, (const float *)u, op.r_off, op.b_off, op.a_off, op.a_log,
                                 op.dt_bias, op.heads, op.groups, op.head_dim, dv, op.q_scale, op.unit_eps, op.state, r.st.req_start,
                                 r.st.slot_ids, r.st.nreq, (float *)mix, (float *)mix + o_floats, T, r.stream));
    ++g_launches;       // the rows' preparation
    RUN(mixers, g_fns.norm_gate((const float *)mix, (const float *)u, op.r_off, op.g_off, op.vec, op.eps, op.heads, dv, op.per_head_norm,
                                op.gate_act, out, r.env.dtype, T, r.stream));
    return JK_OK;
}

int run_embed_pair(Run &r, const RunnerOp &op) {
    JK_REQUIRE(g_fns.embed_pair != nullptr, "runner: an embedding with pairs or a norm needs the blocks module, which was not bound");
    void *out;
    if (int rc = r.slot(op.out_slot, 4LL * r.st.ntok * op.n, &out, "the embedding")) return rc;
    JK_REQUIRE(op.w3 == nullptr || (r.st.slot_ids != nullptr && op.state != nullptr), "runner: pairs of tokens without the requests' last tokens");
    RUN(blocks, g_fns.embed_pair(r.st.tokens, r.st.positions, r.st.row_req, r.st.req_start, r.st.req_pos, r.st.slot_ids, op.w, op.w3, op.w_dtype,
                                 op.buckets, op.mul_prev, op.mul_cur, op.scale, (int *)op.state, op.vec, op.eps, (float *)out, r.st.ntok, op.n, r.stream));
    return JK_OK;
}

int run_join(Run &r, const RunnerOp &op) {
    JK_REQUIRE(g_fns.join_parts != nullptr, "runner: joining sublayers' outputs needs the blocks module, which was not bound");
    const int T = r.st.ntok;
    void *p1, *p2 = nullptr, *p3 = nullptr, *h = nullptr;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.n, &p1, "a sublayer's output")) return rc;
    if (op.in2_slot >= 0)
        if (int rc = r.slot(op.in2_slot, 4LL * T * op.n, &p2, "a second sublayer's output")) return rc;
    if (op.add) {
        if (int rc = r.slot(SLOT_DELTA, 4LL * T * op.n, &p3, "a third sublayer's output")) return rc;
        JK_REQUIRE(!r.pending, "runner: sublayers' outputs join while another product waits to be added");
    } else if (int rc = flush_pending(r, T, op.n)) {
        return rc;
    }
    if (op.out_slot >= 0)
        if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n, &h, "the stream as activations")) return rc;
    RUN(blocks, g_fns.join_parts(r.x(), (const float *)p1, op.vec, op.eps, (const float *)p2, op.vec2, op.eps2, (const float *)p3, h, r.env.dtype, T,
                                 op.n, r.stream));
    return JK_OK;
}

int run_rotate(Run &r, const RunnerOp &op) {
    JK_REQUIRE(g_fns.rotate_rows != nullptr, "runner: a rotation in place needs the mixers module, which was not bound");
    void *u;
    if (int rc = r.slot(op.in_slot, 4LL * r.st.ntok * op.ld, &u, "the rows of a rotation")) return rc;
    RUN(mixers, g_fns.rotate_rows((float *)u, op.ld, op.q_off, op.k_off, op.heads, op.head_dim, op.freq, op.rot_dims, op.rot_half, op.rot_mag,
                                  r.st.positions, r.st.ntok, r.stream));
    return JK_OK;
}

int run_gated_recurrence(Run &r, const RunnerOp &op) {
    JK_REQUIRE(g_fns.gated_recurrence != nullptr, "runner: a gated recurrence needs the blocks module, which was not bound");
    const int T = r.st.ntok, n_pieces = r.st.list_n[op.list_tiles];
    void *u, *y, *out, *scratch = nullptr;
    if (int rc = r.slot(op.in_slot, 4LL * T * op.n, &u, "a recurrence's input")) return rc;
    if (int rc = r.slot(SLOT_TMP, 4LL * T * op.ld, &y, "the projection that holds a recurrence's branch")) return rc;
    if (int rc = r.slot(op.out_slot, (long long)r.elem() * T * op.n, &out, "a recurrence's output")) return rc;
    JK_REQUIRE(r.st.slot_ids != nullptr && op.state != nullptr, "runner: a recurrence without its state slots");
    JK_REQUIRE(op.blocks > 0, "runner: a recurrence in %d parts", op.blocks);
    const int launches = g_fns.gated_recurrence_launches(T, r.st.nreq, op.n / op.blocks, n_pieces);
    const long long floats = launches > 1 ? g_fns.gated_recurrence_scratch(T, op.n, n_pieces) : 0;
    if (floats > 0)
        if (int rc = r.slot(SLOT_SCAN, 4 * floats, &scratch, "a recurrence's pairs and pieces")) return rc;
    RUN(blocks, g_fns.gated_recurrence((const float *)u, op.w, op.w3, op.b1, op.b2, op.decay, (const float *)y + op.g_off, op.ld, op.bias, op.act,
                                       op.state, r.st.req_start, r.st.slot_ids, r.st.nreq, out, r.env.dtype, T, op.n, op.blocks,
                                       r.st.lists[op.list_short], r.st.list_n[op.list_short], r.st.lists[op.list_tiles], n_pieces,
                                       r.st.lists[op.list_aux], r.st.list_n[op.list_aux], (float *)scratch, floats, r.stream));
    g_launches += launches - 1;
    return JK_OK;
}

int run_softcap(Run &r, const RunnerOp &op) {
    if (int rc = need_blocks("a cap on the logits")) return rc;
    const int rows = op.wanted_rows ? r.st.n_want : r.st.ntok;
    if (rows == 0) return JK_OK;
    void *x;
    if (int rc = r.slot(op.in_slot, 4LL * rows * op.n, &x, "the logits")) return rc;
    RUN(blocks, g_fns.softcap((float *)x, op.cap, (long long)rows * op.n, r.stream));
    return JK_OK;
}

}  // namespace

JK_EXPORT int jk_runner_run(const RunnerEnv *envp, const RunnerOp *ops, int first, int count, const RunnerStep *sp,
                            const RunnerBuffers *bp, int flush, cudaStream_t stream) {
    JK_REQUIRE(g_bound, "runner_run: jk_runner_bind has not been called");
    JK_REQUIRE(envp && ops && sp && bp && first >= 0 && count >= 0, "runner_run: an argument is missing");
    JK_REQUIRE(envp->dtype == JK_F32 || envp->dtype == JK_BF16, "runner_run: dtype %d", envp->dtype);
    Run r{*envp, *sp, *bp, stream};
    g_launches = 0;
    const int T = sp->ntok;
    if (T == 0 || count == 0) return JK_OK;
    JK_REQUIRE(bp->slot[SLOT_X] != nullptr, "runner_run: the stream's buffer is missing");
    bool may_fuse = false;
    if (envp->dtype == JK_BF16 && envp->fused_norms && T <= 16 && bp->sumsq != nullptr)
        for (int i = first; i < first + count && !may_fuse; ++i) may_fuse = ops[i].kind == OP_RESIDUAL;
    if (may_fuse) {
        ++g_launches;
        if (cudaMemsetAsync(bp->sumsq, 0, sizeof(unsigned long long) * 16 * (size_t)bp->sumsq_rows, stream) != cudaSuccess)
            JK_FAIL(JK_CUDA_ERROR, "runner: clearing the sums of squares failed");
    }
    FusedNorm fused;              // set by a residual product that took over the norm after it
    int hidden = 0;
    for (int i = first; i < first + count; ++i) {
        const RunnerOp &op = ops[i];
        int rc = JK_OK;
        switch (op.kind) {
            case OP_EMBED:
                hidden = op.n;
                rc = run_embed(r, op);
                break;
            case OP_NORM:
                hidden = op.n;
                if (fused.norm == &op) break;          // the product before did its work
                rc = run_norm(r, op);
                break;
            case OP_QKV: {
                const FusedNorm use = (fused.norm != nullptr && i > first && &ops[i - 1] == fused.norm) ? fused : FusedNorm{};
                rc = run_qkv(r, op, use);
                fused = FusedNorm{};
                break;
            }
            case OP_ATTENTION:
                rc = run_attention(r, op);
                break;
            case OP_RESIDUAL: {
                hidden = op.n;
                const RunnerOp *norm = i + 1 < first + count ? &ops[i + 1] : nullptr;
                const RunnerOp *consumer = i + 2 < first + count ? &ops[i + 2] : nullptr;
                fused = FusedNorm{};
                rc = run_residual(r, op, norm, consumer, i, &fused);
                break;
            }
            case OP_GATE_UP: {
                const FusedNorm use = (fused.norm != nullptr && i > first && &ops[i - 1] == fused.norm) ? fused : FusedNorm{};
                rc = run_gate_up(r, op, use);
                fused = FusedNorm{};
                break;
            }
            case OP_LINEAR: {
                int ran = 0;
                rc = run_linears_together(r, ops, i, first + count, &ran);
                if (rc == JK_OK && ran > 0) i += ran - 1;
                else if (rc == JK_OK) rc = run_linear(r, op);
                break;
            }
            case OP_CAST:
                hidden = op.n;
                rc = run_cast(r, op);
                break;
            case OP_LAYERNORM:
                hidden = op.n;
                rc = run_layernorm(r, op);
                break;
            case OP_CONV_QKV:
                rc = run_conv_qkv(r, op);
                break;
            case OP_LINEAR_ATTENTION:
                rc = run_linear_attention(r, op);
                break;
            case OP_NORM_ADD:
                hidden = op.n;
                rc = run_norm_add(r, op);
                break;
            case OP_REINJECT:
                hidden = op.n;
                rc = run_reinject(r, op);
                break;
            case OP_LATENT_QKV: rc = run_latent_qkv(r, op); break;
            case OP_HEAD_LINEAR: rc = run_head_linear(r, op); break;
            case OP_LATENT_ATTENTION: rc = run_latent_attention(r, op); break;
            case OP_CAUSAL_CONV: rc = run_causal_conv(r, op); break;
            case OP_SELECTIVE_SCAN: rc = run_selective_scan(r, op); break;
            case OP_EXPERTS:
                hidden = op.n;          // with `into_stream` the experts' sum waits for the next norm to add it
                rc = run_experts(r, op);
                break;
            case OP_SOFTCAP: rc = run_softcap(r, op); break;
            case OP_TOKEN_SHIFT: rc = run_token_shift(r, op); break;
            case OP_ACTIVATE: rc = run_activate(r, op); break;
            case OP_ADD_ROWS:
                hidden = op.n;
                rc = run_add_rows(r, op);
                break;
            case OP_DELTA_RULE: rc = run_delta_rule(r, op); break;
            case OP_NORM_PAIR:
                hidden = op.n;
                rc = run_norm_pair(r, op);
                break;
            case OP_EMBED_PAIR:
                hidden = op.n;
                rc = run_embed_pair(r, op);
                break;
            case OP_JOIN:
                hidden = op.n;
                rc = run_join(r, op);
                break;
            case OP_ROTATE: rc = run_rotate(r, op); break;
            case OP_GATED_RECURRENCE: rc = run_gated_recurrence(r, op); break;
            default:
                JK_FAIL(JK_BAD_ARGUMENT, "runner_run: record %d has kind %d", i, op.kind);
        }
        if (rc) return rc;
    }
    // A product that still waits for its addition: a caller that goes on with code of its own (flush) gets a whole stream;
    // at the end of a model nobody reads the stream again.
    if (r.pending && flush) {
        JK_REQUIRE(hidden > 0, "runner_run: a product waits for its addition but no record said how wide the stream is");
        if (int rc = flush_pending(r, T, hidden)) return rc;
    }
    return JK_OK;
}

// How many bytes each slot needs for steps of up to `max_rows` rows with up to `max_want` wanted rows.
JK_EXPORT int jk_runner_slot_bytes(const RunnerEnv *env, const RunnerOp *ops, int count, int max_rows, int max_want, long long *bytes) {
    JK_REQUIRE(env && ops && bytes && max_rows > 0 && max_want >= 0, "runner_slot_bytes: an argument is missing");
    const long long e = env->dtype == JK_F32 ? 4 : 2;
    for (int s = 0; s < RUNNER_SLOTS; ++s) bytes[s] = 0;
    auto need = [&](int slot, long long b) { if (slot >= 0 && slot < RUNNER_SLOTS && b > bytes[slot]) bytes[slot] = b; };
    for (int i = 0; i < count; ++i) {
        const RunnerOp &op = ops[i];
        const long long rows = op.wanted_rows ? max_want : max_rows;
        switch (op.kind) {
            case OP_EMBED: need(op.out_slot, 4 * rows * op.n); break;
            case OP_NORM: need(SLOT_X, 4LL * max_rows * op.n); need(op.out_slot, e * rows * op.n); break;
            case OP_QKV:
                need(op.in_slot, e * rows * op.k); need(op.out_slot, e * rows * op.heads * op.head_dim); need(SLOT_TMP, 4 * rows * op.n);
                break;
            case OP_ATTENTION: {
                need(op.in_slot, e * rows * op.heads * op.head_dim);
                need(op.out_slot, e * rows * op.heads * (op.v_head_dim > 0 ? op.v_head_dim : op.head_dim));
                // the worst step: more rows mean fewer cuts; every context bucket up to the longest
                long long worst = 0;
                for (int context = 256;; context *= 2) {
                    const int c = context < op.max_positions ? context : op.max_positions;
                    for (int n = 1; n <= max_rows; ++n) {
                        const int s = jk::decode_splits(n, op.kv_heads, op.heads / op.kv_heads, jk::decode_keys_hint(c, std::abs(op.window)),
                                                        env->routing.sms, jk::decode_head(op.head_dim, op.v_head_dim));
                        worst = std::max(worst, jk::decode_scratch_floats(n, op.heads, op.v_head_dim > 0 ? op.v_head_dim : op.head_dim, s));
                        if (s <= 1) break;
                    }
                    if (context >= op.max_positions) break;
                }
                need(SLOT_DECODE, 4 * worst);
                break;
            }
            case OP_RESIDUAL: need(op.in_slot, e * rows * op.k); need(SLOT_X, 4 * rows * op.n); need(SLOT_DELTA, 4 * rows * op.n); break;
            case OP_GATE_UP: need(op.in_slot, e * rows * op.k); need(op.out_slot, e * rows * op.n); need(SLOT_TMP, 4 * rows * 2 * op.n); break;
            case OP_LINEAR: need(op.in_slot, e * rows * op.k * (op.in_part + 1)); need(op.out_slot, 4 * rows * (op.ld > 0 ? op.ld : op.n)); break;
            case OP_TOKEN_SHIFT: need(op.in_slot, e * rows * op.n); need(op.out_slot, e * rows * op.n * op.heads); break;
            case OP_ACTIVATE: need(op.in_slot, 4 * rows * (op.ld > 0 ? op.ld : op.n)); need(op.out_slot, e * rows * op.n); break;
            case OP_CAST: need(SLOT_X, 4 * rows * op.n); need(op.out_slot, e * rows * op.n); break;
            case OP_LAYERNORM:
                need(SLOT_X, 4LL * max_rows * op.n); need(op.in_slot, 4 * rows * op.n);
                if (op.out_slot >= 0) need(op.out_slot, e * rows * op.n);
                break;
            case OP_CONV_QKV: need(op.in_slot, 4 * rows * op.ld); need(op.out_slot, e * rows * op.heads * op.head_dim); break;
            case OP_LINEAR_ATTENTION: {
                const long long width = (long long)op.heads * (op.v_head_dim > 0 ? op.v_head_dim : op.head_dim);
                need(op.in_slot, 4 * rows * op.ld); need(SLOT_MIX, 4 * rows * width); need(op.out_slot, e * rows * width);
                if (rows > jk::SCAN_PIECE)
                    need(SLOT_SCAN, 4 * jk::scan_scratch_floats(rows, op.heads, op.head_dim, op.v_head_dim > 0 ? op.v_head_dim : op.head_dim, op.rank > 0));
                break;
            }
            case OP_NORM_ADD:
                need(SLOT_X, 4LL * max_rows * op.n); need(op.in_slot, 4 * rows * op.n);
                if (op.out_slot >= 0) need(op.out_slot, e * rows * op.n);
                if (op.out2_slot >= 0) need(op.out2_slot, e * rows * op.n);
                break;
            case OP_REINJECT: need(SLOT_X, 4 * rows * op.n); need(op.in_slot, 4 * rows * op.n); need(SLOT_ACT, e * rows * op.k); break;
            case OP_LATENT_QKV:
                need(op.in_slot, 4 * rows * op.ld);
                if (op.q_rank > 0) { need(op.out2_slot, e * rows * op.q_rank); break; }
                need(op.out_slot, e * rows * op.heads * (op.rank + op.rot_width));
                need(op.out2_slot, e * rows * op.heads * op.head_dim);
                break;
            case OP_HEAD_LINEAR:
                need(op.in_slot, e * rows * op.heads * op.k); need(op.out_slot, e * rows * op.heads * op.out_hs);
                break;
            case OP_LATENT_ATTENTION: {
                need(op.in_slot, e * rows * op.heads * (op.rank + op.rot_width)); need(op.out_slot, e * rows * op.heads * op.rank);
                long long worst = 0;
                for (int n = 1; n <= 16 && n <= max_rows; ++n)
                    worst = std::max(worst, (long long)n * op.heads * latent_splits(n, op.heads, op.max_positions, env->routing.sms, 128) * (op.rank + 2));
                need(SLOT_DECODE, 4 * worst);
                break;
            }
            case OP_CAUSAL_CONV:
                need(op.in_slot, 4 * rows * op.ld);
                if (op.out_slot >= 0) need(op.out_slot, e * rows * op.n);
                if (op.out2_slot >= 0) need(op.out2_slot, 4 * rows * op.n);
                break;
            case OP_SELECTIVE_SCAN:
                need(op.in_slot, 4 * rows * op.n); need(op.in2_slot, 4 * rows * (op.rank + 2 * op.k)); need(SLOT_TMP, 4 * rows * op.ld);
                need(op.out_slot, e * rows * op.n);
                break;
            case OP_EXPERTS:
                need(op.in_slot, e * rows * op.n); need(SLOT_DELTA, 4 * rows * op.n);
                need(SLOT_ROUTE, 4 * (2LL * (op.experts + op.identity) + 1 + 5 * rows * op.top + rows + 16));
                need(SLOT_ACT, e * rows * op.top * op.ff); need(SLOT_TMP, 4 * rows * op.top * op.n);
                break;
            case OP_SOFTCAP: need(op.in_slot, 4 * rows * op.n); break;
            case OP_NORM_PAIR:
                need(SLOT_X, 4 * rows * op.n); need(op.out_slot, e * rows * op.n);
                if (op.out2_slot >= 0) need(op.out2_slot, e * rows * op.n);
                break;
            case OP_ADD_ROWS: need(SLOT_X, 4 * rows * op.n); break;
            case OP_DELTA_RULE: {
                const long long width = (long long)op.heads * op.v_head_dim;
                const long long per = (op.head_dim + 7) / 8, nper = per <= 4 ? 4 : (per <= 8 ? 8 : (per <= 16 ? 16 : 32));
                need(op.in_slot, 4 * rows * op.ld); need(SLOT_TMP, 4 * rows * op.r_off);
                need(SLOT_SCAN, 4 * ((rows * width + 3) / 4 * 4 + rows * (op.groups * 2 * 8 * nper + 8LL * op.heads)));
                need(op.out_slot, e * rows * width);
                break;
            }
            case OP_EMBED_PAIR: need(op.out_slot, 4 * rows * op.n); break;
            case OP_JOIN:
                need(SLOT_X, 4 * rows * op.n); need(op.in_slot, 4 * rows * op.n);
                if (op.in2_slot >= 0) need(op.in2_slot, 4 * rows * op.n);
                if (op.add) need(SLOT_DELTA, 4 * rows * op.n);
                if (op.out_slot >= 0) need(op.out_slot, e * rows * op.n);
                break;
            case OP_ROTATE: need(op.in_slot, 4 * rows * op.ld); break;
            case OP_GATED_RECURRENCE:
                need(op.in_slot, 4 * rows * op.n); need(SLOT_TMP, 4 * rows * op.ld); need(op.out_slot, e * rows * op.n);
                need(SLOT_SCAN, 4 * 2 * op.n * (rows + jk::scan_max_pieces(rows)));
                break;
            default: JK_FAIL(JK_BAD_ARGUMENT, "runner_slot_bytes: record %d has kind %d", i, op.kind);
        }
    }
    return JK_OK;
}

// Whether records [0, count) can reach a kernel of the tcgen05 product module in a step of up to `max_rows` rows.
JK_EXPORT int jk_runner_needs_gemm_tcgen05(const RunnerEnv *env, const RunnerOp *ops, int count, int max_rows) {
    if (!env || !ops || env->dtype != JK_BF16 || env->routing.library_only) return 0;
    for (int i = 0; i < count; ++i) {
        const RunnerOp &op = ops[i];
        int kind;
        switch (op.kind) {
            case OP_QKV: case OP_LINEAR: case OP_REINJECT: kind = jk::PRODUCT_F32; break;
            case OP_RESIDUAL: kind = jk::PRODUCT_RESIDUAL; break;
            case OP_GATE_UP: kind = jk::PRODUCT_SWIGLU; break;
            default: continue;
        }
        for (int rows : {1, 16, 17, 128, 129, max_rows})
            if (rows <= max_rows || rows == 1) {
                const jk::Route rt = jk::product_route(env->routing, rows, op.n, op.k, kind, true, true);
                if (rt == jk::ROUTE_SKINNY || rt == jk::ROUTE_TCGEN05) return 1;
                // small_ok = true may hide the few-rows kernel behind the small-row one: ask again without it
                const jk::Route rt2 = jk::product_route(env->routing, rows, op.n, op.k, kind, false, true);
                if (rt2 == jk::ROUTE_SKINNY || rt2 == jk::ROUTE_TCGEN05) return 1;
            }
    }
    return 0;
}

// ---- emitters: the records of this architecture's standard parts -----------------------------------------------
static RunnerOp blank(int kind, int in_slot, int out_slot) {
    RunnerOp op;
    memset(&op, 0, sizeof(op));
    op.kind = kind; op.in_slot = in_slot; op.out_slot = out_slot;
    op.scale = 1.f;
    return op;
}

// Causal softmax attention over the paged cache (src/models/jiuge/jiuge.cpp:200-236): the fused q/k/v product with
// rotation and cache write, the attention itself, the output product added into the stream times `residual_scale`.
JK_EXPORT int jk_emit_attention(RunnerOp *out, const void *w_qkv, const float *b_qkv, const void *w_o, int hidden, int heads, int kv_heads,
                                int head_dim, int window, float softmax_scale, float residual_scale, const float *cos_table,
                                const float *sin_table, int interleaved, int max_positions, void *k_pages, void *v_pages, int num_pages,
                                int cache_group, int writes_cache, int list_short, int list_tiles) {
    RunnerOp qkv = blank(OP_QKV, SLOT_H, SLOT_Q);
    qkv.n = (heads + 2 * kv_heads) * head_dim; qkv.k = hidden;
    qkv.heads = heads; qkv.kv_heads = kv_heads; qkv.head_dim = head_dim; qkv.interleaved = interleaved; qkv.writes_cache = writes_cache;
    qkv.cache_group = cache_group; qkv.w = w_qkv; qkv.vec = b_qkv; qkv.cos_table = cos_table; qkv.sin_table = sin_table;
    qkv.k_pages = k_pages; qkv.v_pages = v_pages; qkv.num_pages = num_pages;
    RunnerOp att = blank(OP_ATTENTION, SLOT_Q, SLOT_O);
    att.heads = heads; att.kv_heads = kv_heads; att.head_dim = head_dim; att.window = window; att.softmax_scale = softmax_scale;
    att.cache_group = cache_group; att.list_short = list_short; att.list_tiles = list_tiles; att.max_positions = max_positions;
    att.k_pages = k_pages; att.v_pages = v_pages; att.num_pages = num_pages;
    RunnerOp o = blank(OP_RESIDUAL, SLOT_O, SLOT_X);
    o.n = hidden; o.k = heads * head_dim; o.w = w_o; o.scale = residual_scale;
    out[0] = qkv; out[1] = att; out[2] = o;
    return 3;
}

// SwiGLU feed-forward (src/models/jiuge/jiuge.cpp:247-249): gate | up with the activation, down added into the stream.
JK_EXPORT int jk_emit_swiglu(RunnerOp *out, const void *w_gate_up, const void *w_down, int hidden, int intermediate, float residual_scale) {
    RunnerOp gu = blank(OP_GATE_UP, SLOT_H, SLOT_ACT);
    gu.n = intermediate; gu.k = hidden; gu.w = w_gate_up;
    RunnerOp down = blank(OP_RESIDUAL, SLOT_ACT, SLOT_X);
    down.n = hidden; down.k = intermediate; down.w = w_down; down.scale = residual_scale;
    out[0] = gu; out[1] = down;
    return 2;
}

// RMSNorm over every row (into the next product's activations) or over the wanted rows (the final norm).
JK_EXPORT int jk_emit_rmsnorm(RunnerOp *out, const float *weight, int size, float eps, float out_scale, int wanted_rows) {
    RunnerOp op = blank(OP_NORM, SLOT_X, wanted_rows ? SLOT_HW : SLOT_H);
    op.n = size; op.vec = weight; op.eps = eps; op.scale = out_scale; op.wanted_rows = wanted_rows;
    out[0] = op;
    return 1;
}

JK_EXPORT int jk_emit_embedding(RunnerOp *out, const void *table, int dtype, int hidden, float scale) {
    RunnerOp op = blank(OP_EMBED, -1, SLOT_X);
    op.n = hidden; op.w = table; op.w_dtype = dtype; op.scale = scale;
    out[0] = op;
    return 1;
}

JK_EXPORT int jk_emit_output(RunnerOp *out, const void *w, int vocab, int hidden) {
    RunnerOp op = blank(OP_LINEAR, SLOT_HW, SLOT_LOGITS);
    op.n = vocab; op.k = hidden; op.w = w; op.wanted_rows = 1;
    out[0] = op;
    return 1;
}

// The size of a record, for a caller in another language that mirrors the struct.
JK_EXPORT int jk_runner_op_size() { return (int)sizeof(RunnerOp); }
// sizes[0..4]: RunnerOp, RunnerEnv, RunnerStep, RunnerBuffers, RunnerFns
JK_EXPORT void jk_runner_struct_sizes(int *sizes) {
    sizes[0] = (int)sizeof(RunnerOp); sizes[1] = (int)sizeof(RunnerEnv); sizes[2] = (int)sizeof(RunnerStep);
    sizes[3] = (int)sizeof(RunnerBuffers); sizes[4] = (int)sizeof(RunnerFns);
}
