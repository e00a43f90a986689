// Kernels of blocks whose sublayers sit between two RMS norms, of attention over one small latent vector per token,
// of selective state-space scans and of routed experts:
//
//   norm_add            stream += rmsnorm(sublayer output) * w, and in the same pass the next sublayer's input
//                       rmsnorm(stream) * w'
//   norm_pair           two norms of one stream for two sublayers side by side, the first mixed with the row before it
//   concat_cast         [a | b] side by side as a product's operand; add_bias_rows
//   latent_qkv          queries split into their plain and rotated parts, the latent vector normed, the shared rotated
//                       key part turned, both written into the row's place of the paged cache
//   head_linear         one small product per head (the key and value maps of the latent attention moved to the
//                       query's and the output's side), optionally times a sigmoid gate
//   latent_attention    softmax attention of all heads over one cached row per position, whose leading elements are
//                       the values too; keys may be split among blocks (latent_merge joins them)
//   causal_conv         a short convolution over time per channel with bias and activation, and its tails
//   selective_scan      S <- exp(dt A) S + dt x B, y = S C + D x per channel, with dt = softplus(W low + b) formed here
//   route_topk, route_sort, expert products, expert_combine      experts chosen per token by their scores
//   softcap             cap * tanh(logits / cap)
//   embed_pair          embedding plus a vector per pair of neighbouring tokens, normed
//   join_parts          the outputs of sublayers side by side, each normed or not, added into the stream
//   gated_recurrence    S <- a S + sqrt(1 - a^2) i u per channel with gates from block-diagonal maps of u
//
// Everything that the design wants in float32 is float32 here: norms, angles, scores and softmax weights, routers, the
// scan's state, decays, step sizes and gates.  Products take operands of the activation type T (float or bfloat16) and
// accumulate in float32.  A step's rows are laid out request after request (req_start), continue at req_pos, and keep
// their state in slot slot_ids[request]; a whole prompt, a portion and a single token are one case.
#include "common.cuh"

#include <algorithm>
#include <cstdlib>

JK_DEFINE_ERROR_BUFFER(jk_blocks)

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

enum BlockAct : int { BACT_NONE = 0, BACT_SILU = 1, BACT_GELU_TANH = 2, BACT_SIGMOID = 3, BACT_RELU = 4, BACT_SWISH_CLAMP = 6 };
__device__ __forceinline__ float block_act(int act, float z) {
    switch (act) {
        case BACT_SILU: return silu_f(z);
        case BACT_GELU_TANH: return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
        case BACT_SIGMOID: return sigmoid_f(z);
        case BACT_RELU: return fmaxf(z, 0.f);
        default: return z;
    }
}

// A gated unit's inner value from its two sums g and u and the score s of the row's choice (1 where the score multiplies the
// unit's output instead): act(s g) (s u), or, for BACT_SWISH_CLAMP, with g' = min(g, limit) and u' = clamp(u, -limit, limit),
// g' sigmoid(1.702 g') (u' + 1).
__device__ __forceinline__ float expert_inner(int act, float s, float g, float u, float limit) {
    if (act == BACT_SWISH_CLAMP) {
        g = fminf(s * g, limit);
        u = fminf(fmaxf(s * u, -limit), limit);
        return g * sigmoid_f(1.702f * g) * (u + 1.f);
    }
    return block_act(act, s * g) * (s * u);
}

#define BLOCKS_BY_DTYPE(dtype, name, LAUNCH)                                      \
    do {                                                                          \
        if ((dtype) == JK_F32) { LAUNCH(float); }                                 \
        else if ((dtype) == JK_BF16) { LAUNCH(__nv_bfloat16); }                   \
        else JK_FAIL(JK_UNSUPPORTED, name ": dtype %d", (int)(dtype));            \
    } while (0)

// ---------------------------------------------------------------------------------------------------------------
// x[r] += delta[r] / sqrt(mean(delta[r]^2) + eps) * w;  then, if `out` is given,
// out[r] = T(x[r] / sqrt(mean(x[r]^2) + eps2) * w_next)   (w_next null: out[r] = T(x[r])), and with out2 the same with the weight
// w_next2 (two sublayers side by side read the same stream).
// One block per row; the row stays in shared memory between the passes.
// ---------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16 *p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned *>(&lo); raw.y = *reinterpret_cast<const unsigned *>(&hi);
    *reinterpret_cast<uint2 *>(p) = raw;
}

// VEC: the width is a multiple of four and every operand starts on a 16-byte boundary: four elements move at a time
template <typename T, bool VEC>
__global__ void norm_add_kernel(const float *__restrict__ delta, float *__restrict__ x, const float *__restrict__ w, float eps,
                                const float *__restrict__ w_next, float eps2, T *__restrict__ out, const float *__restrict__ w_next2,
                                T *__restrict__ out2, int d) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float row_buf[];
    __shared__ float scratch[33];
    const size_t base = (size_t)blockIdx.x * d;
    constexpr int S = VEC ? 4 : 1;
    float ss = 0.f;
    for (int c = threadIdx.x * S; c < d; c += blockDim.x * S) {
        if (VEC) {
            const float4 v = *reinterpret_cast<const float4 *>(delta + base + c);
            *reinterpret_cast<float4 *>(row_buf + c) = v;
            ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        } else {
            const float v = delta[base + c];
            row_buf[c] = v;
            ss += v * v;
        }
    }
    const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)d + eps);
    float ss2 = 0.f;
    for (int c = threadIdx.x * S; c < d; c += blockDim.x * S) {
        if (VEC) {
            const float4 xv = *reinterpret_cast<const float4 *>(x + base + c), wv = *reinterpret_cast<const float4 *>(w + c);
            const float4 dv = *reinterpret_cast<const float4 *>(row_buf + c);
            const float4 nx = make_float4(xv.x + dv.x * inv * wv.x, xv.y + dv.y * inv * wv.y, xv.z + dv.z * inv * wv.z, xv.w + dv.w * inv * wv.w);
            *reinterpret_cast<float4 *>(x + base + c) = nx;
            *reinterpret_cast<float4 *>(row_buf + c) = nx;
            ss2 += (nx.x * nx.x + nx.y * nx.y) + (nx.z * nx.z + nx.w * nx.w);
        } else {
            const float nx = x[base + c] + row_buf[c] * inv * w[c];
            x[base + c] = nx;
            row_buf[c] = nx;
            ss2 += nx * nx;
        }
    }
    if (out == nullptr) return;
    const float inv2 = w_next != nullptr ? 1.f / sqrtf(block_sum(ss2, scratch) / (float)d + eps2) : 1.f;
    for (int c = threadIdx.x * S; c < d; c += blockDim.x * S) {
        if (VEC) {
            const float4 v = *reinterpret_cast<const float4 *>(row_buf + c);
            const float4 wv = w_next != nullptr ? *reinterpret_cast<const float4 *>(w_next + c) : make_float4(1.f, 1.f, 1.f, 1.f);
            store4(out + base + c, w_next != nullptr ? make_float4(v.x * inv2 * wv.x, v.y * inv2 * wv.y, v.z * inv2 * wv.z, v.w * inv2 * wv.w) : v);
            if (out2 != nullptr) {
                const float4 w2 = *reinterpret_cast<const float4 *>(w_next2 + c);
                store4(out2 + base + c, make_float4(v.x * inv2 * w2.x, v.y * inv2 * w2.y, v.z * inv2 * w2.z, v.w * inv2 * w2.w));
            }
        } else {
            out[base + c] = from_f32<T>(w_next != nullptr ? row_buf[c] * inv2 * w_next[c] : row_buf[c]);
            if (out2 != nullptr) out2[base + c] = from_f32<T>(row_buf[c] * inv2 * w_next2[c]);
        }
    }
}

JK_EXPORT int jk_norm_add(const float *delta, float *x, const float *w, float eps, const float *w_next, float eps2, void *out,
                          const float *w_next2, void *out2, int dtype, int rows, int d, cudaStream_t stream) {
    if (rows == 0) return JK_OK;
    JK_REQUIRE(delta && x && w && rows > 0 && d > 0, "norm_add: rows %d, width %d", rows, d);
    const size_t smem = (size_t)d * sizeof(float);
    JK_REQUIRE(smem <= 200 * 1024, "norm_add: width %d does not fit shared memory", d);
    JK_REQUIRE(out2 == nullptr || (out && w_next && w_next2), "norm_add: a second norm without the first or without its weight");
    const bool vec = d % 4 == 0 && (uintptr_t)delta % 16 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)w % 16 == 0 &&
                     (w_next == nullptr || (uintptr_t)w_next % 16 == 0) && (out == nullptr || (uintptr_t)out % 16 == 0) &&
                     (uintptr_t)w_next2 % 16 == 0 && (uintptr_t)out2 % 16 == 0;
    // a step of few rows has few blocks: then a thread takes one vector of the row, so that a pass is one round of loads
    int threads = d >= 4096 ? 512 : (d >= 1024 ? 256 : 128);
    if (rows <= 64 && vec) threads = std::min(1024, std::max(threads, (d / 4 + 31) / 32 * 32));
#define LAUNCH_V(T, V)                                                                                                              \
    do {                                                                                                                            \
        if (smem > 46 * 1024) cudaFuncSetAttribute(norm_add_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        jk_launch(norm_add_kernel<T, V>, dim3(rows), dim3(threads), smem, stream, delta, x, w, eps, w_next, eps2, (T *)out, w_next2, (T *)out2, d);   \
    } while (0)
#define LAUNCH(T) if (vec) LAUNCH_V(T, true); else LAUNCH_V(T, false)
    BLOCKS_BY_DTYPE(dtype, "norm_add", LAUNCH);
#undef LAUNCH
#undef LAUNCH_V
    JK_CHECK_LAUNCH("norm_add");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// Two norms of one stream, the first with a token shift: with n_t = x[t] / sqrt(mean(x[t]^2) + eps) * w,
//     h[t]  = T(n_t + (n_(t-1) - n_t) * mu)        (mu null: T(n_t))
//     h2[t] = T(x[t] / sqrt(mean(x[t]^2) + eps2) * w2)        (h2 null: not made)
// n_(t-1) of a portion's first row is the row that the request's last step left (float32; zeros at position 0).  A block takes
// RB rows, asks for all of them and the row ahead of them at once, and adds up their squares in one round.
//
// What is kept of a request is two rows that take turns, state[slot, 2, kept_floats(d)]: n, and behind it (the last word)
// how many positions the sequence had when the row was written.  A step that starts at position p reads the row marked p and
// leaves its last row, marked with the new length, in the other one, so the block with a request's first row and the block
// with its last one never touch the same row (the marks start as 0 and the rows as zeros, which serves position 0).
// ---------------------------------------------------------------------------------------------------------------
struct NormPairArgs {
    const float *x, *w, *mu, *w2;
    float eps, eps2;
    float *state;
    const int *row_req, *req_start, *req_pos, *slot_ids;
    void *h, *h2;
    int T, d;
};

constexpr int NP_THREADS = 512;

__host__ __device__ __forceinline__ int norm_pair_kept_floats(int d) { return (d + 3) / 4 * 4 + 4; }
JK_EXPORT int jk_norm_pair_kept_floats(int d) { return norm_pair_kept_floats(d); }

// Row t in its request: whether it is the first or the last of the step, the kept row it reads (first) and the one it leaves
// (last), and the mark that goes with the latter.  What this reads is read before the block's barrier, the mark written behind it.
struct NormPairRow {
    bool first, last;
    float *from, *to;
    int length;
    __device__ __forceinline__ NormPairRow() : first(false), last(false), from(nullptr), to(nullptr), length(0) {}
    __device__ __forceinline__ NormPairRow(const NormPairArgs &a, int t) : NormPairRow() {
        if (a.mu == nullptr) return;
        const int req = a.row_req[t], start = a.req_start[req], end = a.req_start[req + 1];
        first = start == t;
        last = end == t + 1;
        if (!first && !last) return;
        const int kept = norm_pair_kept_floats(a.d), pos = a.req_pos[req];
        float *base = a.state + (size_t)a.slot_ids[req] * 2 * kept;
        const bool second = *reinterpret_cast<const volatile int *>(base + kept - 1) != pos;      // the other row holds position pos
        from = base + (second ? kept : 0);
        to = base + (second ? 0 : kept);
        length = pos + end - start;
    }
    __device__ __forceinline__ void mark(const NormPairArgs &a) const { reinterpret_cast<int *>(to)[norm_pair_kept_floats(a.d) - 1] = length; }
};

// n sums over a block at once: one barrier, every thread gets all of them.  scratch [n][32]
template <int N>
__device__ __forceinline__ void block_sums(float (&v)[N], float *scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        v[i] = warp_sum(v[i]);
        if (lane == 0) scratch[i * 32 + warp] = v[i];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N; ++i) {
        if (nwarp <= 8) {
            float t = 0.f;
            for (int k = 0; k < nwarp; ++k) t += scratch[i * 32 + k];
            v[i] = t;
        } else {
            v[i] = warp_sum(lane < nwarp ? scratch[i * 32 + lane] : 0.f);
        }
    }
}

__device__ __forceinline__ float sumsq4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }
__device__ __forceinline__ float4 scale4(float4 v, float s, float4 w) { return make_float4(v.x * s * w.x, v.y * s * w.y, v.z * s * w.z, v.w * s * w.w); }
__device__ __forceinline__ float4 mix4(float4 n, float4 before, float4 mu) {
    return make_float4(fmaf(before.x - n.x, mu.x, n.x), fmaf(before.y - n.y, mu.y, n.y), fmaf(before.z - n.z, mu.z, n.z), fmaf(before.w - n.w, mu.w, n.w));
}

// NV vectors of four elements a thread, RB rows a block: few threads with much of a row each, since the sums' shuffles are
// what the kernel would otherwise spend its time on.
template <typename T, int NV, int RB>
__global__ void __launch_bounds__(NP_THREADS) norm_pair_kernel(NormPairArgs a) {
    pdl_trigger();
    __shared__ float scratch[(RB + 1) * 32];
    constexpr bool EARLY = RB == 1;         // few rows: the weights are asked for ahead of the kernel before (no kernel writes them)
    const int n4 = a.d / 4, t0 = blockIdx.x * RB, step = blockDim.x;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    auto load = [&](const float *row, int c) { return row != nullptr && c < n4 ? reinterpret_cast<const float4 *>(row)[c] : zero; };
    float4 w[NV], w2[NV], mu[NV];
    auto load_weights = [&](int i) {
        const int c = threadIdx.x + i * step;
        w[i] = load(a.w, c);
        w2[i] = load(a.h2 != nullptr ? a.w2 : nullptr, c);
        mu[i] = load(a.mu, c);
    };
    if (EARLY) {
#pragma unroll
        for (int i = 0; i < NV; ++i) load_weights(i);
    }
    pdl_wait();
    float4 v[RB + 1][NV];       // v[0]: the row ahead of the block's
#pragma unroll
    for (int r = 0; r <= RB; ++r) {
        const int t = t0 + r - 1;
        const float *row = t < a.T && (r > 0 || (t >= 0 && a.mu != nullptr)) ? a.x + (size_t)t * a.d : nullptr;
#pragma unroll
        for (int i = 0; i < NV; ++i) v[r][i] = load(row, threadIdx.x + i * step);
    }
    NormPairRow at[RB];
#pragma unroll
    for (int r = 0; r < RB; ++r)
        if (t0 + r < a.T) at[r] = NormPairRow(a, t0 + r);
    float ss[RB + 1];
#pragma unroll
    for (int r = 0; r <= RB; ++r) {
        ss[r] = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) ss[r] += sumsq4(v[r][i]);
    }
    block_sums<RB + 1>(ss, scratch);
    float inv2[RB];
#pragma unroll
    for (int r = 0; r <= RB; ++r) {
        const float mean = ss[r] / (float)a.d;
        ss[r] = 1.f / sqrtf(mean + a.eps);
        if (r > 0) inv2[r - 1] = 1.f / sqrtf(mean + a.eps2);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = threadIdx.x + i * step;
        if (c >= n4) continue;
        if (!EARLY) load_weights(i);
        float4 before = scale4(v[0][i], ss[0], w[i]);
#pragma unroll
        for (int r = 0; r < RB; ++r) {
            const int t = t0 + r;
            if (t >= a.T) break;
            if (at[r].first) before = load(at[r].from, c);         // the row that the step before left
            const float4 n = scale4(v[r + 1][i], ss[r + 1], w[i]);
            store4((T *)a.h + (size_t)t * a.d + 4 * c, a.mu != nullptr ? mix4(n, before, mu[i]) : n);
            if (a.h2 != nullptr) store4((T *)a.h2 + (size_t)t * a.d + 4 * c, scale4(v[r + 1][i], inv2[r], w2[i]));
            if (at[r].last) reinterpret_cast<float4 *>(at[r].to)[c] = n;
            before = n;
        }
    }
    if (threadIdx.x == 0) {
#pragma unroll
        for (int r = 0; r < RB; ++r)
            if (at[r].last) at[r].mark(a);
    }
}

// any width and alignment: a block a row, the row before normed once more
template <typename T>
__global__ void __launch_bounds__(NP_THREADS) norm_pair_plain_kernel(NormPairArgs a) {
    pdl_trigger();
    pdl_wait();
    __shared__ float scratch[2 * 32];
    const int t = blockIdx.x;
    const NormPairRow at(a, t);
    const float *x = a.x + (size_t)t * a.d, *xb = a.mu != nullptr && !at.first ? x - a.d : nullptr;
    float ss[2] = {0.f, 0.f};
    for (int c = threadIdx.x; c < a.d; c += blockDim.x) {
        ss[0] += x[c] * x[c];
        if (xb != nullptr) ss[1] += xb[c] * xb[c];
    }
    block_sums<2>(ss, scratch);
    const float mean = ss[0] / (float)a.d, inv = 1.f / sqrtf(mean + a.eps), inv2 = 1.f / sqrtf(mean + a.eps2);
    const float inv_b = 1.f / sqrtf(ss[1] / (float)a.d + a.eps);
    for (int c = threadIdx.x; c < a.d; c += blockDim.x) {
        const float n = x[c] * inv * a.w[c];
        float out = n;
        if (a.mu != nullptr) {
            const float before = xb != nullptr ? xb[c] * inv_b * a.w[c] : at.from[c];
            out = fmaf(before - n, a.mu[c], n);
            if (at.last) at.to[c] = n;
        }
        ((T *)a.h)[(size_t)t * a.d + c] = from_f32<T>(out);
        if (a.h2 != nullptr) ((T *)a.h2)[(size_t)t * a.d + c] = from_f32<T>(x[c] * inv2 * a.w2[c]);
    }
    if (at.last && threadIdx.x == 0) at.mark(a);
}

JK_EXPORT int jk_norm_pair(const float *x, const float *w, const float *mu, float eps, const float *w2, float eps2, float *state,
                           const int *row_req, const int *req_start, const int *req_pos, const int *slot_ids, void *h, void *h2, int dtype,
                           int T, int d, cudaStream_t stream) {
    if (T == 0) return JK_OK;
    JK_REQUIRE(x && w && h && T > 0 && d > 0, "norm_pair: rows %d, width %d", T, d);
    JK_REQUIRE(h2 == nullptr || w2 != nullptr, "norm_pair: a second norm without its weight");
    JK_REQUIRE(mu == nullptr || (state && row_req && req_start && req_pos && slot_ids), "norm_pair: a token shift without its kept rows");
    const bool vec = d % 4 == 0 && d <= 4 * 4 * NP_THREADS && (uintptr_t)x % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)mu % 16 == 0 &&
                     (uintptr_t)w2 % 16 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)h % 16 == 0 && (uintptr_t)h2 % 16 == 0;
    const NormPairArgs a{x, w, mu, w2, eps, eps2, state, row_req, req_start, req_pos, slot_ids, h, h2, T, d};
    // few rows: a thread takes one vector of a row; many: four, and several rows a block (2,048 rows of 2,048 and of 4,096: 9.3
    // and 17.2 us; with one vector a thread and a row a block 19.5 and 47.9)
    const int n4 = (d + 3) / 4;
    const int NV = T <= 64 ? (n4 <= NP_THREADS ? 1 : (n4 <= 2 * NP_THREADS ? 2 : 4)) : (n4 <= 64 ? 1 : (n4 <= 128 ? 2 : 4));
    const int threads = vec ? std::max(64, ((n4 + NV - 1) / NV + 31) / 32 * 32) : std::max(64, std::min(NP_THREADS, (d + 31) / 32 * 32));
    const int RB = T >= 4 * 148 ? 4 : (T >= 2 * 148 ? 2 : 1);
    const dim3 grid((T + RB - 1) / RB);
#define LAUNCH_NV(TT, V)                                                                        \
    if (RB == 4) jk_launch(norm_pair_kernel<TT, V, 4>, grid, dim3(threads), 0, stream, a);      \
    else if (RB == 2) jk_launch(norm_pair_kernel<TT, V, 2>, grid, dim3(threads), 0, stream, a); \
    else jk_launch(norm_pair_kernel<TT, V, 1>, grid, dim3(threads), 0, stream, a)
#define LAUNCH(TT)                                                                           \
    if (!vec) jk_launch(norm_pair_plain_kernel<TT>, dim3(T), dim3(threads), 0, stream, a);   \
    else if (NV == 1) { LAUNCH_NV(TT, 1); }                                                  \
    else if (NV == 2) { LAUNCH_NV(TT, 2); }                                                  \
    else { LAUNCH_NV(TT, 4); }
    BLOCKS_BY_DTYPE(dtype, "norm_pair", LAUNCH);
#undef LAUNCH
#undef LAUNCH_NV
    JK_CHECK_LAUNCH("norm_pair");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// out[t] = T([a[t] | b[t]]): two float32 streams side by side as the operand of one product.
// ---------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void concat_cast_kernel(const float *__restrict__ a, const float *__restrict__ b, T *__restrict__ out, int d, size_t total) {
    pdl_trigger();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / (2 * d);
        const int c = (int)(i % (2 * d));
        out[i] = from_f32<T>(c < d ? a[t * d + c] : b[t * d + c - d]);
    }
}

JK_EXPORT int jk_concat_cast(const float *a, const float *b, void *out, int dtype, int rows, int d, cudaStream_t stream) {
    if (rows == 0) return JK_OK;
    JK_REQUIRE(a && b && out && rows > 0 && d > 0, "concat_cast: rows %d, width %d", rows, d);
    const size_t total = (size_t)rows * 2 * d;
    const int blocks = (int)std::min<size_t>((total + 255) / 256, 148 * 16);
#define LAUNCH(T) jk_launch(concat_cast_kernel<T>, dim3(blocks), dim3(256), 0, stream, a, b, (T *)out, d, total)
    BLOCKS_BY_DTYPE(dtype, "concat_cast", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("concat_cast");
    return JK_OK;
}

__global__ void add_bias_rows_kernel(float *__restrict__ x, const float *__restrict__ bias, int d, size_t total) {
    pdl_trigger();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) x[i] += bias[i % d];
}

JK_EXPORT int jk_add_bias_rows(float *x, const float *bias, int rows, int d, cudaStream_t stream) {
    if (rows == 0) return JK_OK;
    JK_REQUIRE(x && bias && rows > 0 && d > 0, "add_bias_rows: rows %d, width %d", rows, d);
    const size_t total = (size_t)rows * d;
    const int blocks = (int)std::min<size_t>((total + 255) / 256, 148 * 16);
    jk_launch(add_bias_rows_kernel, dim3(blocks), dim3(256), 0, stream, x, bias, d, total);
    JK_CHECK_LAUNCH("add_bias_rows");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// Queries and cache rows of the latent attention, from the float32 rows u [T, ld] of one fused product:
//   u[t, q_off + h (dn + dr) + e]      head h of the query: dn plain elements, then dr that are rotated
//   u[t, kv_off + e]                   e < R: the latent vector before its norm; then dr elements of the shared key part
// Rotation of the first `rot_dims` of the dr elements in pairs (2i, 2i+1) (rot_half: (i, i + rot_dims / 2)) by p * freq[i],
// formed in float32, with cos and sin times `mag`.  kv_off < 0: the queries only; a query latent (q_norm_w): the cache row and
// the query latent only.  Out: q_plain [T, H dn] (the operand of the per-head product that moves the key map to the query),
// the rotated parts into q_full [T, H, R + dr] behind the R elements which that product fills, and the cache row of the
// position, [latent * norm weight / rms | rotated key part], into pages [pages, page_size, R + dr].  One block per row.
// ---------------------------------------------------------------------------------------------------------------
struct LatentQkvArgs {
    const float *u;
    int ld, q_off, kv_off, H, dn, dr, R, rot_dims;
    const float *freq;
    float mag, eps;
    const float *norm_w;
    const int *positions, *row_req, *block_table;
    int max_blocks, page_size;
    void *q_plain, *q_full, *pages;
    const float *q_norm_w;      // with it: q_plain [T, q_rank] = rmsnorm(u[q_off .. q_off + q_rank)) * q_norm_w, the queries' own latent
    int q_rank;                 // vector (the heads' queries are then a product of it, made by the records that follow)
    int rot_half;
};

// element e of a part whose first rot_dims elements are rotated (src: the part's elements)
__device__ __forceinline__ float latent_rotated(const LatentQkvArgs &a, const float *src, int e, float fpos) {
    const float val = src[e];
    if (e >= a.rot_dims) return val;
    const int half = a.rot_dims >> 1;
    const bool first = a.rot_half ? e < half : !(e & 1);
    const int pair = a.rot_half ? (first ? e : e - half) : e >> 1;
    const float other = src[a.rot_half ? (first ? e + half : e - half) : e ^ 1];
    float sn, cs;
    sincosf(fpos * a.freq[pair], &sn, &cs);
    sn *= a.mag; cs *= a.mag;
    return first ? fmaf(val, cs, -other * sn) : fmaf(val, cs, other * sn);
}

template <typename T>
__global__ void latent_qkv_kernel(LatentQkvArgs a) {
    pdl_trigger();
    pdl_wait();
    __shared__ float scratch[33];
    const int t = blockIdx.x;
    const float *u = a.u + (size_t)t * a.ld;
    const int pos = a.positions[t];
    const float fpos = (float)pos;
    const int dq = a.dn + a.dr, D = a.R + a.dr;
    // the latent vector's norm
    T *crow = nullptr;
    if (a.kv_off >= 0) {
        float ss = 0.f;
        for (int e = threadIdx.x; e < a.R; e += blockDim.x) {
            const float v = u[a.kv_off + e];
            ss += v * v;
        }
        const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)a.R + a.eps);
        const int page = a.block_table[(size_t)a.row_req[t] * a.max_blocks + pos / a.page_size];
        crow = (T *)a.pages + ((size_t)page * a.page_size + (size_t)(pos % a.page_size)) * D;
        for (int e = threadIdx.x; e < a.R; e += blockDim.x) crow[e] = from_f32<T>(u[a.kv_off + e] * inv * a.norm_w[e]);
    }
    if (a.q_norm_w != nullptr) {
        float sq = 0.f;
        for (int e = threadIdx.x; e < a.q_rank; e += blockDim.x) {
            const float v = u[a.q_off + e];
            sq += v * v;
        }
        const float inv_q = 1.f / sqrtf(block_sum(sq, scratch) / (float)a.q_rank + a.eps);
        for (int e = threadIdx.x; e < a.q_rank; e += blockDim.x)
            ((T *)a.q_plain)[(size_t)t * a.q_rank + e] = from_f32<T>(u[a.q_off + e] * inv_q * a.q_norm_w[e]);
        for (int e = threadIdx.x; e < a.dr; e += blockDim.x) crow[a.R + e] = from_f32<T>(latent_rotated(a, u + a.kv_off + a.R, e, fpos));
        return;
    }
    // rotated parts: every head's query part and (head index H) the shared key part
    for (int idx = threadIdx.x; idx < (a.kv_off >= 0 ? a.H + 1 : a.H) * a.dr; idx += blockDim.x) {
        const int h = idx / a.dr, e = idx % a.dr;
        const float val = latent_rotated(a, h == a.H ? u + a.kv_off + a.R : u + a.q_off + (size_t)h * dq + a.dn, e, fpos);
        if (h == a.H) crow[a.R + e] = from_f32<T>(val);
        else ((T *)a.q_full)[((size_t)t * a.H + h) * D + a.R + e] = from_f32<T>(val);
    }
    for (int idx = threadIdx.x; idx < a.H * a.dn; idx += blockDim.x) {
        const int h = idx / a.dn, e = idx % a.dn;
        ((T *)a.q_plain)[(size_t)t * a.H * a.dn + idx] = from_f32<T>(u[a.q_off + (size_t)h * dq + e]);
    }
}

JK_EXPORT int jk_latent_qkv(const float *u, int ld, int q_off, int kv_off, int H, int dn, int dr, int R, int rot_dims, const float *freq,
                            float mag, const float *norm_w, float eps, const int *positions, const int *row_req, const int *block_table,
                            int max_blocks, int page_size, void *q_plain, void *q_full, void *pages, int dtype, int T,
                            const float *q_norm_w, int q_rank, int rot_half, cudaStream_t stream) {
    if (T == 0) return JK_OK;
    JK_REQUIRE(u && positions && row_req && q_plain && (q_full || q_norm_w), "latent_qkv: an argument is missing");
    JK_REQUIRE(kv_off < 0 || (norm_w && block_table && pages), "latent_qkv: a cache row without its pages");
    JK_REQUIRE(q_norm_w == nullptr || (q_rank > 0 && kv_off >= 0), "latent_qkv: a query latent of %d elements without the keys' latent", q_rank);
    JK_REQUIRE(H > 0 && dn >= 0 && dr >= 0 && R > 0 && page_size > 0, "latent_qkv: heads %d, sizes %d + %d, latent %d", H, dn, dr, R);
    JK_REQUIRE(rot_dims >= 0 && rot_dims <= dr && rot_dims % 2 == 0 && (rot_dims == 0 || freq), "latent_qkv: rotation of %d of %d elements", rot_dims, dr);
    LatentQkvArgs a{u, ld, q_off, kv_off, H, dn, dr, R, rot_dims, freq, mag, eps, norm_w, positions, row_req, block_table,
                    max_blocks, page_size, q_plain, q_full, pages, q_norm_w, q_rank, rot_half};
    const int work = q_norm_w ? std::max(q_rank, R) : H * (dn + dr);
    const int threads = work >= 2048 ? 512 : (work >= 512 ? 256 : 128);
#define LAUNCH(TT) jk_launch(latent_qkv_kernel<TT>, dim3(T), dim3(threads), 0, stream, a)
    BLOCKS_BY_DTYPE(dtype, "latent_qkv", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("latent_qkv");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// Tiled products: C[M, N] = A[M, K] W[N, K]^T with float32 accumulation, operands of type T.  A block of 256 threads
// makes a tile of 64 x 64.  float operands: on the CUDA cores (FFMA in the order of K, a thread 4 x 4 of the tile, K
// through shared memory 16 at a time).  bfloat16 operands: on the tensor cores (mma.sync m16n8k16, a warp 16 x 32 of the
// tile, K through shared memory 32 at a time by asynchronous copies three tiles deep, fragments by ldmatrix).  Rows of A may be picked through an index (a_rows).
// With GLU a second weight tile W2 runs along and the epilogue sees both sums.  A thread holds 16 sums; tile_at() says
// where sum e lies in the tile.  Used per head (head_linear) and per expert (expert products), where the problem depends
// on the block.
// ---------------------------------------------------------------------------------------------------------------
constexpr int GT_M = 64, GT_N = 64, GT_K = 16;

template <typename T> struct OnTensorCores { static constexpr bool value = false; };
template <> struct OnTensorCores<__nv_bfloat16> { static constexpr bool value = true; };

template <typename T>
__device__ __forceinline__ void tile_at(int e, int *row, int *col) {
    if (OnTensorCores<T>::value) {
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
        *row = (warp & 3) * 16 + (lane >> 2) + ((e & 2) ? 8 : 0);
        *col = (warp >> 2) * 32 + (e >> 2) * 8 + (lane & 3) * 2 + (e & 1);
    } else {
        *row = (threadIdx.x / 16) * 4 + e / 4;
        *col = (threadIdx.x % 16) * 4 + e % 4;
    }
}

template <bool GLU>
__device__ __forceinline__ void tile_product(const float *__restrict__ A, size_t lda, const int *__restrict__ a_rows, int M,
                                             const float *__restrict__ W, const float *__restrict__ W2, size_t ldw, int N, int K, int m0, int n0,
                                             float (&acc)[16], float (&acc2)[16]) {
    __shared__ float As[GT_K][GT_M + 4];
    __shared__ float Ws[GT_K][GT_N + 4];
    __shared__ float W2s[GLU ? GT_K : 1][GT_N + 4];
    const int tid = threadIdx.x, ty = tid / 16, tx = tid % 16;
    const int lr = tid / 4, lk = (tid % 4) * 4;      // this thread loads row lr, k lk .. lk + 3 of each operand tile
    const int am = m0 + lr, wn = n0 + lr;
    const float *arow = am < M ? A + (size_t)(a_rows ? a_rows[am] : am) * lda : nullptr;
    const float *wrow = wn < N ? W + (size_t)wn * ldw : nullptr;
    const float *w2row = (GLU && wn < N) ? W2 + (size_t)wn * ldw : nullptr;
#pragma unroll
    for (int e = 0; e < 16; ++e) { acc[e] = 0.f; acc2[e] = 0.f; }
    for (int k0 = 0; k0 < K; k0 += GT_K) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int k = k0 + lk + i;
            As[lk + i][lr] = (arow && k < K) ? arow[k] : 0.f;
            Ws[lk + i][lr] = (wrow && k < K) ? wrow[k] : 0.f;
            if (GLU) W2s[lk + i][lr] = (w2row && k < K) ? w2row[k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < GT_K; ++k) {
            float av[4], wv[4], w2v[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { av[i] = As[k][ty * 4 + i]; wv[i] = Ws[k][tx * 4 + i]; if (GLU) w2v[i] = W2s[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i * 4 + j] = fmaf(av[i], wv[j], acc[i * 4 + j]);
                    if (GLU) acc2[i * 4 + j] = fmaf(av[i], w2v[j], acc2[i * 4 + j]);
                }
        }
        __syncthreads();
    }
}

__device__ __forceinline__ void ldmatrix_x4(unsigned &r0, unsigned &r1, unsigned &r2, unsigned &r3, const void *smem_row) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(smem_row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];\n" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16_16816(float *d, unsigned a0, unsigned a1, unsigned a2, unsigned a3, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

constexpr int TC_K = 32, TC_LD = TC_K + 8;     // rows of 80 bytes: 16-byte aligned for ldmatrix, and eight of them hit distinct banks

// eight elements of a row from k on; zeros beyond K or where there is no row
__device__ __forceinline__ uint4 fetch8(const __nv_bfloat16 *row, int k, int K, bool vec) {
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (row != nullptr) {
        if (vec && k + 8 <= K) {
            v = *reinterpret_cast<const uint4 *>(row + k);
        } else {
            __nv_bfloat16 t[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) t[i] = k + i < K ? row[k + i] : __float2bfloat16_rn(0.f);
            v = *reinterpret_cast<const uint4 *>(t);
        }
    }
    return v;
}

// eight elements of a row from k on into shared memory, zeros beyond K or where there is no row: an asynchronous 16-byte
// copy where rows are 16-byte aligned, else element by element
__device__ __forceinline__ void stage8(__nv_bfloat16 *dst, const __nv_bfloat16 *row, int k, int K, bool vec) {
    if (vec) {
        const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
        const int left = row != nullptr ? K - k : 0;
        const int bytes = left >= 8 ? 16 : (left > 0 ? 2 * left : 0);
        const __nv_bfloat16 *src = bytes > 0 ? row + k : dst;          // nothing is read when bytes is 0; the address only has to be one
        if (bytes > 0) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(src), "r"(bytes) : "memory");
        else *reinterpret_cast<uint4 *>(dst) = make_uint4(0u, 0u, 0u, 0u);
    } else {
        *reinterpret_cast<uint4 *>(dst) = fetch8(row, k, K, false);
    }
}

constexpr int TC_STAGES = 3;        // tiles of K in flight: a block keeps 2 x 5 KB (or 3 x with GLU) a stage on its way

template <bool GLU>
__device__ __forceinline__ void tile_product(const __nv_bfloat16 *__restrict__ A, size_t lda, const int *__restrict__ a_rows, int M,
                                             const __nv_bfloat16 *__restrict__ W, const __nv_bfloat16 *__restrict__ W2, size_t ldw, int N, int K,
                                             int m0, int n0, float (&acc)[16], float (&acc2)[16]) {
    __shared__ __align__(16) __nv_bfloat16 As[TC_STAGES][GT_M * TC_LD];
    __shared__ __align__(16) __nv_bfloat16 Ws[TC_STAGES][GT_N * TC_LD];
    __shared__ __align__(16) __nv_bfloat16 W2s[GLU ? TC_STAGES : 1][GLU ? GT_N * TC_LD : 8];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int lr = tid / 4, lk = (tid % 4) * 8;      // this thread stages row lr, k lk .. lk + 7 of each operand tile
    const int am = m0 + lr, wn = n0 + lr;
    const __nv_bfloat16 *arow = am < M ? A + (size_t)(a_rows ? a_rows[am] : am) * lda : nullptr;
    const __nv_bfloat16 *wrow = wn < N ? W + (size_t)wn * ldw : nullptr;
    const __nv_bfloat16 *w2row = (GLU && wn < N) ? W2 + (size_t)wn * ldw : nullptr;
    const bool vec_a = lda % 8 == 0 && (uintptr_t)A % 16 == 0;
    const bool vec_w = ldw % 8 == 0 && (uintptr_t)W % 16 == 0 && (!GLU || (uintptr_t)W2 % 16 == 0);
#pragma unroll
    for (int e = 0; e < 16; ++e) { acc[e] = 0.f; acc2[e] = 0.f; }
    const int a_row = (warp & 3) * 16 + (lane & 15), a_col = (lane >> 4) * 8;
    const int b_row = (warp >> 2) * 32 + (lane >> 4) * 8 + (lane & 7), b_col = ((lane >> 3) & 1) * 8;
    const int nk = (K + TC_K - 1) / TC_K;
    auto stage = [&](int kt) {          // tile kt of K into its buffer; a group is committed even when there is no such tile
        if (kt < nk) {
            const int b = kt % TC_STAGES, k = kt * TC_K + lk;
            stage8(As[b] + lr * TC_LD + lk, arow, k, K, vec_a);
            stage8(Ws[b] + lr * TC_LD + lk, wrow, k, K, vec_w);
            if (GLU) stage8(W2s[b] + lr * TC_LD + lk, w2row, k, K, vec_w);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
#pragma unroll
    for (int i = 0; i < TC_STAGES - 1; ++i) stage(i);
    for (int kt = 0; kt < nk; ++kt) {
        asm volatile("cp.async.wait_group %0;\n" ::"n"(TC_STAGES - 2) : "memory");       // tile kt has landed (for this thread)
        __syncthreads();                                                                  // ... and for all; the buffer of tile kt - 1 is free
        stage(kt + TC_STAGES - 1);
        const __nv_bfloat16 *as = As[kt % TC_STAGES], *ws = Ws[kt % TC_STAGES], *w2s = W2s[GLU ? kt % TC_STAGES : 0];
#pragma unroll
        for (int kk = 0; kk < TC_K; kk += 16) {
            unsigned a0, a1, a2, a3;
            ldmatrix_x4(a0, a1, a2, a3, as + a_row * TC_LD + kk + a_col);
#pragma unroll
            for (int p = 0; p < 2; ++p) {          // two tiles of eight columns at a time
                unsigned b0, b1, b2, b3;
                ldmatrix_x4(b0, b1, b2, b3, ws + (b_row + p * 16) * TC_LD + kk + b_col);
                mma_bf16_16816(acc + (2 * p) * 4, a0, a1, a2, a3, b0, b1);
                mma_bf16_16816(acc + (2 * p + 1) * 4, a0, a1, a2, a3, b2, b3);
                if (GLU) {
                    ldmatrix_x4(b0, b1, b2, b3, w2s + (b_row + p * 16) * TC_LD + kk + b_col);
                    mma_bf16_16816(acc2 + (2 * p) * 4, a0, a1, a2, a3, b0, b1);
                    mma_bf16_16816(acc2 + (2 * p + 1) * 4, a0, a1, a2, a3, b2, b3);
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();        // a second product of the same block may stage at once
}

// C = A W^T for a float32 A and a bfloat16 W on the tensor cores without rounding A: every element of A is cut into two
// bfloat16 halves (a = hi + lo, which keeps 16 bits of its mantissa) and both halves meet the same weights.  With TWO a second
// weight tile runs along.  The next step of K is on its way in registers while the tensor cores work on this one.
template <bool TWO>
__device__ __forceinline__ void tile_product_split(const float *__restrict__ A, size_t lda, int M, const __nv_bfloat16 *__restrict__ W,
                                                   const __nv_bfloat16 *__restrict__ W2, size_t ldw, int N, int K, int m0, int n0,
                                                   float (&acc)[16], float (&acc2)[16]) {
    __shared__ __align__(16) __nv_bfloat16 Ah[GT_M * TC_LD];
    __shared__ __align__(16) __nv_bfloat16 Al[GT_M * TC_LD];
    __shared__ __align__(16) __nv_bfloat16 Ws[GT_N * TC_LD];
    __shared__ __align__(16) __nv_bfloat16 W2s[TWO ? GT_N * TC_LD : 8];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int lr = tid / 4, lk = (tid % 4) * 8;
    const int am = m0 + lr, wn = n0 + lr;
    const float *arow = am < M ? A + (size_t)am * lda : nullptr;
    const __nv_bfloat16 *wrow = wn < N ? W + (size_t)wn * ldw : nullptr;
    const __nv_bfloat16 *w2row = (TWO && wn < N) ? W2 + (size_t)wn * ldw : nullptr;
    const bool vec_w = ldw % 8 == 0 && (uintptr_t)W % 16 == 0 && (!TWO || (uintptr_t)W2 % 16 == 0);
    const bool vec_a = lda % 4 == 0 && (uintptr_t)A % 16 == 0;
#pragma unroll
    for (int e = 0; e < 16; ++e) { acc[e] = 0.f; acc2[e] = 0.f; }
    const int a_row = (warp & 3) * 16 + (lane & 15), a_col = (lane >> 4) * 8;
    const int b_row = (warp >> 2) * 32 + (lane >> 4) * 8 + (lane & 7), b_col = ((lane >> 3) & 1) * 8;
    __align__(16) float av[8];
    uint4 wv, w2v = make_uint4(0u, 0u, 0u, 0u);
    auto fetch = [&](int k0) {
        if (vec_a && arow != nullptr && k0 + lk + 8 <= K) {
            *reinterpret_cast<float4 *>(av) = *reinterpret_cast<const float4 *>(arow + k0 + lk);
            *reinterpret_cast<float4 *>(av + 4) = *reinterpret_cast<const float4 *>(arow + k0 + lk + 4);
        } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) av[i] = (arow != nullptr && k0 + lk + i < K) ? arow[k0 + lk + i] : 0.f;
        }
        wv = fetch8(wrow, k0 + lk, K, vec_w);
        if (TWO) w2v = fetch8(w2row, k0 + lk, K, vec_w);
    };
    fetch(0);
    for (int k0 = 0; k0 < K; k0 += TC_K) {
        __align__(16) __nv_bfloat16 h8[8], l8[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            h8[i] = __float2bfloat16_rn(av[i]);
            l8[i] = __float2bfloat16_rn(av[i] - __bfloat162float(h8[i]));
        }
        *reinterpret_cast<uint4 *>(Ah + lr * TC_LD + lk) = *reinterpret_cast<const uint4 *>(h8);
        *reinterpret_cast<uint4 *>(Al + lr * TC_LD + lk) = *reinterpret_cast<const uint4 *>(l8);
        *reinterpret_cast<uint4 *>(Ws + lr * TC_LD + lk) = wv;
        if (TWO) *reinterpret_cast<uint4 *>(W2s + lr * TC_LD + lk) = w2v;
        __syncthreads();
        if (k0 + TC_K < K) fetch(k0 + TC_K);
#pragma unroll
        for (int kk = 0; kk < TC_K; kk += 16) {
            unsigned h0, h1, h2, h3, l0, l1, l2, l3;
            ldmatrix_x4(h0, h1, h2, h3, Ah + a_row * TC_LD + kk + a_col);
            ldmatrix_x4(l0, l1, l2, l3, Al + a_row * TC_LD + kk + a_col);
#pragma unroll
            for (int p = 0; p < 2; ++p) {
                unsigned b0, b1, b2, b3;
                ldmatrix_x4(b0, b1, b2, b3, Ws + (b_row + p * 16) * TC_LD + kk + b_col);
                mma_bf16_16816(acc + (2 * p) * 4, l0, l1, l2, l3, b0, b1);
                mma_bf16_16816(acc + (2 * p + 1) * 4, l0, l1, l2, l3, b2, b3);
                mma_bf16_16816(acc + (2 * p) * 4, h0, h1, h2, h3, b0, b1);
                mma_bf16_16816(acc + (2 * p + 1) * 4, h0, h1, h2, h3, b2, b3);
                if (TWO) {
                    ldmatrix_x4(b0, b1, b2, b3, W2s + (b_row + p * 16) * TC_LD + kk + b_col);
                    mma_bf16_16816(acc2 + (2 * p) * 4, l0, l1, l2, l3, b0, b1);
                    mma_bf16_16816(acc2 + (2 * p + 1) * 4, l0, l1, l2, l3, b2, b3);
                    mma_bf16_16816(acc2 + (2 * p) * 4, h0, h1, h2, h3, b0, b1);
                    mma_bf16_16816(acc2 + (2 * p + 1) * 4, h0, h1, h2, h3, b2, b3);
                }
            }
        }
        __syncthreads();
    }
}

// out[t, h * out_hs + n] = T(sum_k in[t, h * K + k] * w[h, n, k]) (* sigmoid(gate[t * gate_ld + h * N + n]), or with gate_head
// sigmoid(gate[t * gate_ld + h]))
template <typename T>
__global__ void __launch_bounds__(256) head_linear_kernel(const T *__restrict__ in, const T *__restrict__ w, T *__restrict__ out, int rows, int H,
                                                          int N, int K, int out_hs, const float *__restrict__ gate, int gate_ld, int gate_head) {
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.z, m0 = blockIdx.x * GT_M, n0 = blockIdx.y * GT_N;
    float acc[16], unused[16];
    tile_product<false>(in + (size_t)h * K, (size_t)H * K, nullptr, rows, w + (size_t)h * N * K, (const T *)nullptr, (size_t)K, N, K, m0, n0, acc, unused);
#pragma unroll
    for (int e = 0; e < 16; ++e) {
        int r, c;
        tile_at<T>(e, &r, &c);
        const int t = m0 + r, n = n0 + c;
        if (t >= rows || n >= N) continue;
        float v = acc[e];
        if (gate != nullptr) v *= sigmoid_f(gate[(size_t)t * gate_ld + (gate_head ? (size_t)h : (size_t)h * N + n)]);
        out[((size_t)t * H + h) * out_hs + n] = from_f32<T>(v);
    }
}

JK_EXPORT int jk_head_linear(const void *in, const void *w, void *out, int dtype, int rows, int H, int N, int K, int out_hs,
                             const float *gate, int gate_ld, int gate_head, cudaStream_t stream) {
    if (rows == 0) return JK_OK;
    JK_REQUIRE(in && w && out && rows > 0 && H > 0 && N > 0 && K > 0 && out_hs >= N, "head_linear: rows %d, heads %d, %d x %d into %d", rows, H, N, K, out_hs);
    JK_REQUIRE(H <= 65535, "head_linear: %d heads exceed one launch", H);
    dim3 grid((rows + GT_M - 1) / GT_M, (N + GT_N - 1) / GT_N, H);
#define LAUNCH(T) jk_launch(head_linear_kernel<T>, grid, dim3(256), 0, stream, (const T *)in, (const T *)w, (T *)out, rows, H, N, K, out_hs, gate, gate_ld, gate_head)
    BLOCKS_BY_DTYPE(dtype, "head_linear", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("head_linear");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// Attention of H heads over one cached row per position: row j of a request is [c_j (R) | r_j (dr)]; a query row of a
// head is [a (R) | b (dr)]; score = (a . c_j + b . r_j) * scale over j <= position; out = sum_j softmax_j c_j  [R].
// A block takes one query row and LA_WARPS heads; 32 cached rows at a time pass shared memory (read once for all the
// block's heads), a lane takes one of them for the scores and a slice of R for the weighted sum.  Scores, the running
// maximum, the weights and the sums are float32.  With `splits` > 1 the keys of a row are cut into that many ranges
// (blockIdx.z); a range leaves its unnormalised sum, maximum and normaliser in `part` and latent_merge joins them.
// ---------------------------------------------------------------------------------------------------------------
constexpr int LA_WARPS = 8;

struct LatentAttnArgs {
    const void *q, *pages;
    void *out;
    float *part;            // [T, H, splits, R + 2]
    const int *positions, *row_req, *block_table;
    int T, H, R, dr, page_size, max_blocks, splits;
    float scale;
    int window;             // the mask as one number (jk_mask_lo): 0 every earlier key, W > 0 the last W keys
    const float *sink_w;    // [H] or null: one more key per softmax, of this score and without a value
};

// what a sink adds to the normaliser that belongs to the maximum m
__device__ __forceinline__ float latent_sink(const float *sink_w, int h, float m) { return sink_w != nullptr ? expf(sink_w[h] - m) : 0.f; }

template <typename T, int NS>
__global__ void __launch_bounds__(LA_WARPS * 32) latent_attention_kernel(LatentAttnArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float la_smem[];
    const int D = a.R + a.dr, DP = D + 1;
    float *qs = la_smem;                                  // [LA_WARPS][D]
    float *tile = la_smem + LA_WARPS * D;                 // [32][D + 1]
    __shared__ long long row_off[32];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t = blockIdx.y, h = blockIdx.x * LA_WARPS + warp;
    const bool active = h < a.H;
    const int pos = a.positions[t];
    const int *bt = a.block_table + (size_t)a.row_req[t] * a.max_blocks;
    int lo = jk_mask_lo(pos, a.window), hi = pos + 1;
    if (a.splits > 1) {
        const int chunk = (((hi - lo + a.splits - 1) / a.splits) + 31) / 32 * 32;
        lo += blockIdx.z * chunk;
        hi = min(pos + 1, lo + chunk);
    }
    if (active) {
        const T *qrow = (const T *)a.q + ((size_t)t * a.H + h) * D;
        for (int e = lane; e < D; e += 32) qs[warp * D + e] = to_f32(qrow[e]);
    }
    float m = -INFINITY, l = 0.f;
    float acc[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) acc[i] = 0.f;
    const T *pages = (const T *)a.pages;
    for (int j0 = lo; j0 < hi; j0 += 32) {
        const int n = min(32, hi - j0);
        if (threadIdx.x < 32) {
            const int j = j0 + threadIdx.x;
            row_off[threadIdx.x] = threadIdx.x < n ? ((long long)bt[j / a.page_size] * a.page_size + (j % a.page_size)) * D : -1;
        }
        __syncthreads();
        for (int idx = threadIdx.x; idx < n * D; idx += blockDim.x) {
            const int r = idx / D, e = idx % D;
            tile[r * DP + e] = to_f32(pages[row_off[r] + e]);
        }
        __syncthreads();
        if (active) {
            float s = -INFINITY;
            if (lane < n) {
                const float *kr = tile + lane * DP, *qr = qs + warp * D;
                float dot = 0.f;
                for (int e = 0; e < D; ++e) dot = fmaf(qr[e], kr[e], dot);
                s = dot * a.scale;
            }
            const float m_new = fmaxf(m, warp_max(s));
            const float p = lane < n ? expf(s - m_new) : 0.f;
            const float corr = expf(m - m_new);
            l = l * corr + warp_sum(p);
            m = m_new;
#pragma unroll
            for (int i = 0; i < NS; ++i) acc[i] *= corr;
            for (int jj = 0; jj < n; ++jj) {
                const float pj = __shfl_sync(0xffffffffu, p, jj);
                const float *vr = tile + jj * DP;
#pragma unroll
                for (int i = 0; i < NS; ++i) {
                    const int e = lane + 32 * i;
                    if (e < a.R) acc[i] = fmaf(pj, vr[e], acc[i]);
                }
            }
        }
        __syncthreads();
    }
    if (!active) return;
    if (a.splits > 1) {
        float *p = a.part + (((size_t)t * a.H + h) * a.splits + blockIdx.z) * (a.R + 2);
#pragma unroll
        for (int i = 0; i < NS; ++i) {
            const int e = lane + 32 * i;
            if (e < a.R) p[e] = acc[i];
        }
        if (lane == 0) { p[a.R] = m; p[a.R + 1] = l; }
        return;
    }
    T *orow = (T *)a.out + ((size_t)t * a.H + h) * a.R;
    const float inv = 1.f / (l + latent_sink(a.sink_w, h, m));
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int e = lane + 32 * i;
        if (e < a.R) orow[e] = from_f32<T>(acc[i] * inv);
    }
}

// one block per (row, head): the ranges' sums brought to one maximum and added in the order of the ranges.  The ranges'
// factors exp(m_s - M) / l are formed once by the first warp (a lane a range) and kept in shared memory; a thread then
// takes columns, with all ranges' loads of a column asked for before the sum starts.
constexpr int LM_THREADS = 128, LM_MAX_SPLITS = 64;

template <typename T>
__global__ void __launch_bounds__(LM_THREADS) latent_merge_kernel(const float *__restrict__ part, T *__restrict__ out, int H, int R, int splits,
                                                                  const float *__restrict__ sink_w) {
    pdl_trigger();
    pdl_wait();
    __shared__ float factor[LM_MAX_SPLITS];
    const int lane = threadIdx.x & 31, idx = blockIdx.x;
    const float *p = part + (size_t)idx * splits * (R + 2);
    if (threadIdx.x < 32) {
        float ms[LM_MAX_SPLITS / 32], ls[LM_MAX_SPLITS / 32];
        float M = -INFINITY;
#pragma unroll
        for (int i = 0; i < LM_MAX_SPLITS / 32; ++i) {
            const int s = lane + 32 * i;
            ms[i] = s < splits ? p[(size_t)s * (R + 2) + R] : -INFINITY;
            ls[i] = s < splits ? p[(size_t)s * (R + 2) + R + 1] : 0.f;
            M = fmaxf(M, ms[i]);
        }
        M = warp_max(M);
        float l = 0.f;
#pragma unroll
        for (int i = 0; i < LM_MAX_SPLITS / 32; ++i) {
            ms[i] = ms[i] > -INFINITY ? expf(ms[i] - M) : 0.f;
            l += ls[i] * ms[i];
        }
        l = warp_sum(l) + latent_sink(sink_w, idx % H, M);
        const float inv = 1.f / l;
#pragma unroll
        for (int i = 0; i < LM_MAX_SPLITS / 32; ++i) {
            const int s = lane + 32 * i;
            if (s < splits) factor[s] = ms[i] * inv;
        }
    }
    __syncthreads();
    for (int e = threadIdx.x; e < R; e += LM_THREADS) {
        float v = 0.f;
        int s = 0;
        for (; s + 8 <= splits; s += 8) {
            float t[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) t[i] = p[(size_t)(s + i) * (R + 2) + e];
#pragma unroll
            for (int i = 0; i < 8; ++i) v = fmaf(t[i], factor[s + i], v);
        }
        for (; s < splits; ++s) v = fmaf(p[(size_t)s * (R + 2) + e], factor[s], v);
        out[(size_t)idx * R + e] = from_f32<T>(v);
    }
}

// The same attention on the tensor cores (bfloat16, mma.sync m16n8k16 with float32 accumulation).  Since every head reads
// the same cached rows, (query row, head) pairs are the M side of the products: a block of eight warps takes 32 pairs of
// one request (RT rows x HT heads) and walks the request's cached rows 32 at a time through shared memory.  Warp (mw, nw)
// has pairs mw * 16 .. + 15; for the scores it takes the tile's keys nw * 8 .. + 7 over the whole row width, the four nw
// warps exchange scores through shared memory, every thread forms the softmax weights of its own fragment (float32; the
// maximum and the sum go around the four lanes that share a row), and for the weighted sum it owns the output columns
// nw * NT * 8 .. of all 32 keys, the cached tile serving as the value operand through ldmatrix.trans.  Tiles of cached
// rows arrive by asynchronous copies into two buffers that take turns.  Ranges as above.
constexpr int LT_PAIRS = 32, LT_KEYS = 32;

struct LatentTcArgs {
    const __nv_bfloat16 *q, *pages;
    __nv_bfloat16 *out;
    float *part;
    const int *positions, *req_start, *block_table;
    int nreq, H, R, dr, page_size, max_blocks, splits, HT, RT, ldk;
    float scale;
    int buffers;        // 2: the tile after the one at work is on its way; 1: where two would leave an SM room for one block only
    int window;         // the mask as one number (jk_mask_lo)
    const float *sink_w;    // as above
};

__device__ __forceinline__ void ldmatrix_x2(unsigned &r0, unsigned &r1, const void *smem_row) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(smem_row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];\n" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned &r0, unsigned &r1, unsigned &r2, unsigned &r3, const void *smem_row) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(smem_row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];\n" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const unsigned *>(&v);
}

template <int NT>       // tiles of eight output columns per warp
__global__ void __launch_bounds__(256) latent_attention_tc_kernel(LatentTcArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char lt_smem[];
    // the block's request and rows
    int req = -1, t0 = 0, nrows = 0;
    {
        int tiles = 0;
        for (int i = 0; i < a.nreq; ++i) {
            const int len = a.req_start[i + 1] - a.req_start[i];
            const int mine = (len + a.RT - 1) / a.RT;
            if ((int)blockIdx.x < tiles + mine) {
                const int local = ((int)blockIdx.x - tiles) * a.RT;
                req = i; t0 = a.req_start[i] + local; nrows = min(a.RT, len - local);
                break;
            }
            tiles += mine;
        }
    }
    if (req < 0) return;
    const int h0 = blockIdx.y * a.HT;
    const int D = a.R + a.dr, DP = (D + 15) / 16 * 16, LDK = a.ldk, LDQ = DP + 8;
    __nv_bfloat16 *Qs = reinterpret_cast<__nv_bfloat16 *>(lt_smem);                 // [32][LDQ]
    __nv_bfloat16 *Kbuf = Qs + LT_PAIRS * LDQ;                                      // two tiles of [32][LDK] that take turns
    float *Sb = reinterpret_cast<float *>(Kbuf + a.buffers * LT_KEYS * LDK);        // [2][16][33]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, mw = warp & 1, nw = warp >> 1;
    const bool vec = D % 8 == 0 && (uintptr_t)a.pages % 16 == 0 && (uintptr_t)a.q % 16 == 0;
    {
        const int q8 = LDQ / 8;
        for (int idx = tid; idx < LT_PAIRS * q8; idx += 256) {
            const int p = idx / q8, e = (idx % q8) * 8, r = p / a.HT, h = h0 + p % a.HT;
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (r < nrows && h < a.H && e < D) {
                const __nv_bfloat16 *src = a.q + ((size_t)(t0 + r) * a.H + h) * D + e;
                if (vec && e + 8 <= D) {
                    v = *reinterpret_cast<const uint4 *>(src);
                } else {
                    __nv_bfloat16 tmp[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) tmp[i] = e + i < D ? src[i] : __float2bfloat16_rn(0.f);
                    v = *reinterpret_cast<const uint4 *>(tmp);
                }
            }
            *reinterpret_cast<uint4 *>(Qs + p * LDQ + e) = v;
        }
    }
    const int max_pos = a.positions[t0 + nrows - 1];
    int lo = jk_mask_lo(a.positions[t0], a.window), hi = max_pos + 1;       // positions rise along a request's rows
    if (a.splits > 1) {
        const int chunk = (((hi - lo + a.splits - 1) / a.splits) + 31) / 32 * 32;
        lo += blockIdx.z * chunk;
        hi = min(max_pos + 1, lo + chunk);
    }
    // this thread's two rows of its warp's 16 pairs
    const int pa = mw * 16 + (lane >> 2), pb = pa + 8;
    const int ra = pa / a.HT, rb = pb / a.HT, ha = h0 + pa % a.HT, hb = h0 + pb % a.HT;
    const bool va = ra < nrows && ha < a.H, vb = rb < nrows && hb < a.H;
    const int pos_a = va ? a.positions[t0 + ra] : -1, pos_b = vb ? a.positions[t0 + rb] : -1;
    const int lo_a = jk_mask_lo(pos_a, a.window), lo_b = jk_mask_lo(pos_b, a.window);
    float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
    const int *bt = a.block_table + (size_t)req * a.max_blocks;
    // A tile of cached rows into one of the two buffers: 16-byte asynchronous copies (zeros where there is no row or no
    // column) when rows are multiples of 16 bytes, else element by element.  The tile after the one at work is always
    // on its way.
    auto fetch_tile = [&](int j0, __nv_bfloat16 *Ks) {
        const int n = min(LT_KEYS, hi - j0);
        const __nv_bfloat16 *src_row[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {           // a warp brings rows warp, warp + 8, ...; their places first, then the copies
            const int r = warp + 8 * i, j = r < n ? j0 + r : lo;
            src_row[i] = a.pages + ((size_t)bt[j / a.page_size] * a.page_size + (size_t)(j % a.page_size)) * D;
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = warp + 8 * i;
            __nv_bfloat16 *dst_row = Ks + r * LDK;
            for (int c = lane * 8; c < LDK; c += 256) {
                const bool there = r < n && c < D;
                if (vec) {
                    const unsigned d = (unsigned)__cvta_generic_to_shared(dst_row + c);
                    const int bytes = there ? 16 : 0;
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(src_row[i] + (there ? c : 0)), "r"(bytes) : "memory");
                } else {
                    __nv_bfloat16 tmp[8];
#pragma unroll
                    for (int e = 0; e < 8; ++e) tmp[e] = (there && c + e < D) ? src_row[i][c + e] : __float2bfloat16_rn(0.f);
                    *reinterpret_cast<uint4 *>(dst_row + c) = *reinterpret_cast<const uint4 *>(tmp);
                }
            }
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    const bool two = a.buffers > 1;
    if (lo < hi && two) fetch_tile(lo, Kbuf);
    int turn = 0;
    for (int j0 = lo; j0 < hi; j0 += LT_KEYS, turn ^= (two ? 1 : 0)) {
        const int n = min(LT_KEYS, hi - j0);
        const __nv_bfloat16 *Ks = Kbuf + turn * LT_KEYS * LDK;
        if (!two) {
            fetch_tile(j0, Kbuf);
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        } else if (j0 + LT_KEYS < hi) {
            fetch_tile(j0 + LT_KEYS, Kbuf + (turn ^ 1) * LT_KEYS * LDK);
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        // scores of this warp's pairs against the keys nw * 8 .. + 7
        float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};      // two chains of sums that take turns
        {
            const __nv_bfloat16 *qp = Qs + (mw * 16 + (lane & 15)) * LDQ + (lane >> 4) * 8;
            const __nv_bfloat16 *kp = Ks + (nw * 8 + (lane & 7)) * LDK + ((lane >> 3) & 1) * 8;
            int kk = 0;
            for (; kk + 32 <= DP; kk += 32) {
                unsigned a0, a1, a2, a3, b0, b1, c0, c1, c2, c3, d0, d1;
                ldmatrix_x4(a0, a1, a2, a3, qp + kk);
                ldmatrix_x2(b0, b1, kp + kk);
                ldmatrix_x4(c0, c1, c2, c3, qp + kk + 16);
                ldmatrix_x2(d0, d1, kp + kk + 16);
                mma_bf16_16816(s, a0, a1, a2, a3, b0, b1);
                mma_bf16_16816(s2, c0, c1, c2, c3, d0, d1);
            }
            if (kk < DP) {
                unsigned a0, a1, a2, a3, b0, b1;
                ldmatrix_x4(a0, a1, a2, a3, qp + kk);
                ldmatrix_x2(b0, b1, kp + kk);
                mma_bf16_16816(s, a0, a1, a2, a3, b0, b1);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) s[i] += s2[i];
        }
        {
            float *row_a = Sb + (mw * 16 + (lane >> 2)) * 33, *row_b = row_a + 8 * 33;
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                const int k = nw * 8 + (lane & 3) * 2 + c, j = j0 + k;
                row_a[k] = (k < n && j <= pos_a && j >= lo_a) ? s[c] * a.scale : -INFINITY;
                row_b[k] = (k < n && j <= pos_b && j >= lo_b) ? s[2 + c] * a.scale : -INFINITY;
            }
        }
        __syncthreads();
        // softmax weights of this thread's fragment: keys (lane & 3) * 2 + {0, 1} + {0, 8, 16, 24} of its two rows
        float pa_[8], pb_[8];
        {
            const float *row_a = Sb + (mw * 16 + (lane >> 2)) * 33, *row_b = row_a + 8 * 33;
            float mx_a = -INFINITY, mx_b = -INFINITY;
#pragma unroll
            for (int g = 0; g < 4; ++g)
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const int k = g * 8 + (lane & 3) * 2 + c;
                    pa_[g * 2 + c] = row_a[k]; pb_[g * 2 + c] = row_b[k];
                    mx_a = fmaxf(mx_a, pa_[g * 2 + c]); mx_b = fmaxf(mx_b, pb_[g * 2 + c]);
                }
            mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 1)); mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 2));
            mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 1)); mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 2));
            const float mn_a = fmaxf(m_a, mx_a), mn_b = fmaxf(m_b, mx_b);
            const float corr_a = mn_a == -INFINITY ? 1.f : expf(m_a - mn_a), corr_b = mn_b == -INFINITY ? 1.f : expf(m_b - mn_b);
            float sum_a = 0.f, sum_b = 0.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                pa_[i] = mn_a == -INFINITY ? 0.f : expf(pa_[i] - mn_a);
                pb_[i] = mn_b == -INFINITY ? 0.f : expf(pb_[i] - mn_b);
                sum_a += pa_[i]; sum_b += pb_[i];
            }
            sum_a += __shfl_xor_sync(0xffffffffu, sum_a, 1); sum_a += __shfl_xor_sync(0xffffffffu, sum_a, 2);
            sum_b += __shfl_xor_sync(0xffffffffu, sum_b, 1); sum_b += __shfl_xor_sync(0xffffffffu, sum_b, 2);
            l_a = l_a * corr_a + sum_a; l_b = l_b * corr_b + sum_b;
            m_a = mn_a; m_b = mn_b;
#pragma unroll
            for (int i = 0; i < NT; ++i) { o[i][0] *= corr_a; o[i][1] *= corr_a; o[i][2] *= corr_b; o[i][3] *= corr_b; }
        }
        // weighted sum: keys 0 .. 15, then 16 .. 31; values = the cached rows' columns nw * NT * 8 ..
#pragma unroll
        for (int ks = 0; ks < 2; ++ks) {
            const unsigned a0 = pack_bf16(pa_[ks * 4 + 0], pa_[ks * 4 + 1]), a1 = pack_bf16(pb_[ks * 4 + 0], pb_[ks * 4 + 1]);
            const unsigned a2 = pack_bf16(pa_[ks * 4 + 2], pa_[ks * 4 + 3]), a3 = pack_bf16(pb_[ks * 4 + 2], pb_[ks * 4 + 3]);
#pragma unroll
            for (int i = 0; i < NT; i += 2) {
                unsigned b0, b1, b2, b3;
                ldmatrix_x4_trans(b0, b1, b2, b3, Ks + (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDK + (nw * NT + i) * 8 + (lane >> 4) * 8);
                mma_bf16_16816(o[i], a0, a1, a2, a3, b0, b1);
                mma_bf16_16816(o[i + 1], a0, a1, a2, a3, b2, b3);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const bool valid = half ? vb : va;
        if (!valid) continue;
        const int t = t0 + (half ? rb : ra), h = half ? hb : ha;
        const float l = half ? l_b : l_a, m = half ? m_b : m_a;
        if (a.splits > 1) {
            float *p = a.part + (((size_t)t * a.H + h) * a.splits + blockIdx.z) * (a.R + 2);
#pragma unroll
            for (int i = 0; i < NT; ++i)
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const int col = (nw * NT + i) * 8 + (lane & 3) * 2 + c;
                    if (col < a.R) p[col] = o[i][half * 2 + c];
                }
            if (nw == 0 && (lane & 3) == 0) { p[a.R] = m; p[a.R + 1] = l; }
        } else {
            __nv_bfloat16 *orow = a.out + ((size_t)t * a.H + h) * a.R;
            const float inv = 1.f / (l + latent_sink(a.sink_w, h, m));
#pragma unroll
            for (int i = 0; i < NT; ++i)
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const int col = (nw * NT + i) * 8 + (lane & 3) * 2 + c;
                    if (col < a.R) orow[col] = __float2bfloat16_rn(o[i][half * 2 + c] * inv);
                }
        }
    }
}

static bool latent_tc_enabled() {
    static const bool on = [] { const char *e = std::getenv("JK_LATENT_NO_TC"); return !(e && e[0] == '1'); }();
    return on;
}

// floats of `part` that `splits` ranges of T rows need
JK_EXPORT long long jk_latent_attention_scratch(int T, int H, int R, int splits) {
    return splits > 1 ? (long long)T * H * splits * (R + 2) : 0;
}

// `req_start` [nreq + 1] (may be null): with it, bfloat16 rows go to the tensor-core kernel (latent sizes up to 512).
JK_EXPORT int jk_latent_attention(const void *q, const void *pages, void *out, float *part, int dtype, const int *positions,
                                  const int *row_req, const int *block_table, int max_blocks, int page_size, int T, int H, int R,
                                  int dr, float scale, int splits, const int *req_start, int nreq, int window, const float *sink_w,
                                  cudaStream_t stream) {
    if (T == 0) return JK_OK;
    JK_REQUIRE(window >= 0, "latent_attention: window %d", window);
    JK_REQUIRE(q && pages && out && positions && row_req && block_table, "latent_attention: an argument is missing");
    JK_REQUIRE(H > 0 && R > 0 && dr >= 0 && page_size > 0 && max_blocks > 0, "latent_attention: heads %d, latent %d + %d", H, R, dr);
    JK_REQUIRE(R <= 1024, "latent_attention: a latent size of %d exceeds 1024", R);
    JK_REQUIRE(T <= 65535, "latent_attention: %d rows exceed one launch (65535)", T);
    if (splits < 1) splits = 1;
    JK_REQUIRE(splits == 1 || part != nullptr, "latent_attention: split keys need room for their parts");
    JK_REQUIRE(splits <= LM_MAX_SPLITS, "latent_attention: %d ranges exceed %d", splits, LM_MAX_SPLITS);
    const int D = R + dr;
    if (dtype == JK_BF16 && req_start != nullptr && nreq > 0 && R <= 512 && latent_tc_enabled()) {
        int HT = 1;
        while (HT * 2 <= std::min(H, LT_PAIRS)) HT *= 2;
        const int RT = LT_PAIRS / HT, tiles8 = (R + 7) / 8, per = (tiles8 + 3) / 4;
        const int NT = per <= 2 ? 2 : (per <= 4 ? 4 : (per <= 8 ? 8 : 16));
        const int DP = (D + 15) / 16 * 16, ldk = std::max(DP, 4 * NT * 8) + 8;
        // two tile buffers unless that leaves an SM (about 227 KB, 1 KB a block reserved) room for one block where one buffer leaves
        // room for two and the launch has more blocks than SMs
        const size_t fixed = (size_t)LT_PAIRS * (DP + 8) * 2 + 2 * 16 * 33 * sizeof(float), tile = (size_t)LT_KEYS * ldk * 2;
        dim3 grid((T + RT - 1) / RT + nreq, (H + HT - 1) / HT, splits);
        static const int sms = [] { int n = 148, dev = 0; cudaGetDevice(&dev); cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev); return n; }();
        const bool second_block_fits = fixed + 2 * tile > 112 * 1024 && fixed + tile <= 112 * 1024;
        const int buffers = (second_block_fits && (long long)((T + RT - 1) / RT) * grid.y * grid.z > sms) ? 1 : 2;
        LatentTcArgs ta{(const __nv_bfloat16 *)q, (const __nv_bfloat16 *)pages, (__nv_bfloat16 *)out, part, positions, req_start, block_table,
                        nreq, H, R, dr, page_size, max_blocks, splits, HT, RT, ldk, scale, buffers, window, sink_w};
        const size_t smem_tc = fixed + buffers * tile;
        JK_REQUIRE(grid.y <= 65535, "latent_attention: %d heads", H);
#define LAUNCH_TC(NT_)                                                                                                                       \
    do {                                                                                                                                    \
        if (smem_tc > 46 * 1024) cudaFuncSetAttribute(latent_attention_tc_kernel<NT_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_tc); \
        jk_launch(latent_attention_tc_kernel<NT_>, grid, dim3(256), smem_tc, stream, ta);                                                   \
    } while (0)
        if (NT == 2) LAUNCH_TC(2); else if (NT == 4) LAUNCH_TC(4); else if (NT == 8) LAUNCH_TC(8); else LAUNCH_TC(16);
#undef LAUNCH_TC
        JK_CHECK_LAUNCH("latent_attention_tc");
        if (splits > 1) {
            const int n = T * H;
            jk_launch(latent_merge_kernel<__nv_bfloat16>, dim3(n), dim3(LM_THREADS), 0, stream, (const float *)part, (__nv_bfloat16 *)out, H, R, splits, sink_w);
            JK_CHECK_LAUNCH("latent_merge");
        }
        return JK_OK;
    }
    LatentAttnArgs a{q, pages, out, part, positions, row_req, block_table, T, H, R, dr, page_size, max_blocks, splits, scale, window, sink_w};
    const size_t smem = ((size_t)LA_WARPS * D + 32 * (size_t)(D + 1)) * sizeof(float);
    JK_REQUIRE(smem <= 220 * 1024, "latent_attention: rows of %d elements do not fit shared memory", D);
    dim3 grid((H + LA_WARPS - 1) / LA_WARPS, T, splits);
#define LAUNCH_NS(TT, NS)                                                                                                                   \
    do {                                                                                                                                    \
        if (smem > 46 * 1024) cudaFuncSetAttribute(latent_attention_kernel<TT, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        jk_launch(latent_attention_kernel<TT, NS>, grid, dim3(LA_WARPS * 32), smem, stream, a);                                             \
    } while (0)
#define LAUNCH(TT)                                  \
    if (R <= 64) LAUNCH_NS(TT, 2);                  \
    else if (R <= 128) LAUNCH_NS(TT, 4);            \
    else if (R <= 256) LAUNCH_NS(TT, 8);            \
    else if (R <= 512) LAUNCH_NS(TT, 16);           \
    else LAUNCH_NS(TT, 32)
    BLOCKS_BY_DTYPE(dtype, "latent_attention", LAUNCH);
#undef LAUNCH
#undef LAUNCH_NS
    JK_CHECK_LAUNCH("latent_attention");
    if (splits > 1) {
        const int n = T * H;
#define LAUNCH(TT) jk_launch(latent_merge_kernel<TT>, dim3(n), dim3(LM_THREADS), 0, stream, (const float *)part, (TT *)out, H, R, splits, sink_w)
        BLOCKS_BY_DTYPE(dtype, "latent_merge", LAUNCH);
#undef LAUNCH
        JK_CHECK_LAUNCH("latent_merge");
    }
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// A short causal convolution over time on each of C channels, with bias and activation:
//     y_t[c] = act(bias[c] + sum_j taps[c, j] * u_(t - J + 1 + j)[c])          zeros before the sequence starts
// u is a column range of float32 rows [T, ld], with in_bias[c] added (the projection's bias; not before the sequence starts).  The
// J - 1 rows before a portion come from the request's tail [slots, J - 1, C] (s = J - 2 the newest; in_bias included), which moves
// forward: that of a request with one row in the step in the row's own pass (a channel is one thread's), the others' by conv_tails.  y goes out as float32 (what a
// recurrence reads) and in the activation type (what a product reads).
// ---------------------------------------------------------------------------------------------------------------
struct ConvArgs {
    const float *u;
    int ld, off, C, J, act;
    const float *taps, *bias;
    float *tail;
    const int *row_req, *req_start, *slot_ids;
    float *y32;
    void *yT;
    const float *in_bias;
};

template <typename T>
__global__ void causal_conv_kernel(ConvArgs a, int rows) {
    pdl_trigger();
    pdl_wait();
    const size_t total = (size_t)rows * a.C;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const int t = (int)(i / a.C), c = (int)(i % a.C);
        const int req = a.row_req[t];
        const int back = t - a.req_start[req];
        float *tail = a.J > 1 ? a.tail + (size_t)a.slot_ids[req] * (a.J - 1) * a.C : nullptr;
        float acc = a.bias ? a.bias[c] : 0.f, uv = 0.f;
        const float in_bias = a.in_bias ? a.in_bias[c] : 0.f;
        for (int j = 0; j < a.J; ++j) {
            const int d = a.J - 1 - j;          // rows back
            uv = d <= back ? a.u[(size_t)(t - d) * a.ld + a.off + c] + in_bias : tail[(size_t)(a.J - 1 + back - d) * a.C + c];
            acc = fmaf(a.taps[(size_t)c * a.J + j], uv, acc);
        }
        if (tail != nullptr && a.req_start[req + 1] - a.req_start[req] == 1) {
            for (int s = 0; s + 2 < a.J; ++s) tail[(size_t)s * a.C + c] = tail[(size_t)(s + 1) * a.C + c];
            tail[(size_t)(a.J - 2) * a.C + c] = uv;          // the row's own input
        }
        const float y = block_act(a.act, acc);
        if (a.y32) a.y32[i] = y;
        if (a.yT) ((T *)a.yT)[i] = from_f32<T>(y);
    }
}

// tail[slot, s, c] <- the input J - 1 - s rows before the end of the request's sequence after this step; a thread owns
// (request, channel) and reads every old entry before it overwrites it
__global__ void conv_tails_kernel(ConvArgs a, int nreq) {
    pdl_trigger();
    pdl_wait();
    const int idx = blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= nreq * a.C) return;
    const int req = idx / a.C, c = idx % a.C;
    const int first = a.req_start[req], n = a.req_start[req + 1] - first;
    if (n == 1) return;         // moved forward by the row's own thread
    float *tail = a.tail + (size_t)a.slot_ids[req] * (a.J - 1) * a.C;
    const float in_bias = a.in_bias ? a.in_bias[c] : 0.f;
    for (int s = 0; s < a.J - 1; ++s) {
        const int off = n - (a.J - 1) + s;
        const float v = off >= 0 ? a.u[(size_t)(first + off) * a.ld + a.off + c] + in_bias : tail[(size_t)(s + n) * a.C + c];
        tail[(size_t)s * a.C + c] = v;
    }
}

JK_EXPORT int jk_causal_conv(const float *u, int ld, int off, int C, const float *taps, const float *bias, int J, int act, float *tail,
                             const int *row_req, const int *req_start, const int *slot_ids, float *y32, void *yT, int dtype, int T,
                             int nreq, const float *in_bias, cudaStream_t stream) {
    if (T == 0) return JK_OK;
    JK_REQUIRE(u && taps && row_req && req_start && C > 0 && J >= 1 && (y32 || yT), "causal_conv: an argument is missing");
    JK_REQUIRE(J == 1 || (tail && slot_ids), "causal_conv: %d taps without the tails' state", J);
    ConvArgs a{u, ld, off, C, J, act, taps, bias, tail, row_req, req_start, slot_ids, y32, yT, in_bias};
    const size_t total = (size_t)T * C;
    const int blocks = (int)std::min<size_t>((total + 255) / 256, 148 * 16);
#define LAUNCH(TT) jk_launch(causal_conv_kernel<TT>, dim3(blocks), dim3(256), 0, stream, a, T)
    BLOCKS_BY_DTYPE(dtype, "causal_conv", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("causal_conv");
    if (J > 1 && T > nreq) {
        jk_launch(conv_tails_kernel, dim3((nreq * C + 127) / 128), dim3(128), 0, stream, a, nreq);
        JK_CHECK_LAUNCH("conv_tails");
    }
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// Selective scan.  Per request, channel c of E and state n of N, over the request's rows in order:
//     dt_t[c]  = softplus(sum_k Wdt[c, k] low_t[k] + bdt[c])                low_t = [dt part (K) | B_t (N) | C_t (N)]
//     S[c, n] <- exp(dt_t[c] A[c, n]) S[c, n] + dt_t[c] x_t[c] B_t[n]
//     y_t[c]   = sum_n S[c, n] C_t[n] + Dskip[c] x_t[c];   out_t[c] = T(y_t[c] * silu(z_t[c]))
// all float32; S lives in state[slot, c, n] between steps.  Eight neighbouring lanes share a channel: lane `part` keeps
// the states part, part + 8, ... in registers.  A block of 128 threads owns 16 channels of one request and walks the
// request's rows.
// ---------------------------------------------------------------------------------------------------------------
constexpr int SS_LANES = 8, SS_THREADS = 128, SS_CHANNELS = SS_THREADS / SS_LANES, SS_CHUNK = 32;

struct ScanArgs {
    const float *x;         // [T, E] after convolution and activation
    const float *low;       // [T, ld_low]
    int ld_low, K, N, E;
    const float *z;         // z_t[c] = z[t * ld_z + c]
    int ld_z;
    const void *Wdt;        // [E, K] in the activation type (float32 mode: float; bfloat16 mode: as the checkpoint stores it)
    const float *bdt, *A, *Dskip;
    float *state;
    const int *req_start, *slot_ids;
    void *out;
    const float *dt;        // step sizes made ahead, dt[t * ld_dt + c], or null: they are formed while the rows are staged
    int ld_dt;
};

// dt[t, c] = softplus(low[t, :K] . Wdt[c] + bdt[c]) ahead of the scan, as one product: float32 weights on the CUDA
// cores; bfloat16 weights (as a 16-bit checkpoint stores them) on the tensor cores with the float32 rows cut in two
// halves, so that nothing of them is rounded away.  The sums and the softplus are float32.
template <typename TW>
__global__ void __launch_bounds__(256) scan_steps_kernel(const float *__restrict__ low, int ld_low, const TW *__restrict__ Wdt,
                                                         const float *__restrict__ bdt, float *__restrict__ dt, int ld_dt, int rows, int E, int K) {
    pdl_trigger();
    pdl_wait();
    const int m0 = blockIdx.x * GT_M, n0 = blockIdx.y * GT_N;
    float acc[16], unused[16];
    if constexpr (OnTensorCores<TW>::value) {
        tile_product_split<false>(low, (size_t)ld_low, rows, Wdt, (const TW *)nullptr, (size_t)K, E, K, m0, n0, acc, unused);
    } else {
        tile_product<false>(low, (size_t)ld_low, nullptr, rows, Wdt, (const float *)nullptr, (size_t)K, E, K, m0, n0, acc, unused);
    }
#pragma unroll
    for (int e = 0; e < 16; ++e) {
        int r, c;
        tile_at<TW>(e, &r, &c);
        const int t = m0 + r, ch = n0 + c;
        if (t < rows && ch < E) dt[(size_t)t * ld_dt + ch] = softplus_f(acc[e] + bdt[ch]);
    }
}

// Rows pass shared memory SS_CHUNK at a time (step sizes, inputs, B and C staged by all threads), so a row of the
// recurrence costs no global load and no exchange between lanes: a lane leaves its share of a row's sum in shared
// memory, and a chunk's outputs are added up and leave together, times silu(z).
template <typename T, int NPER>
__global__ void __launch_bounds__(SS_THREADS) selective_scan_kernel(ScanArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float ss_smem[];
    float *s_dt = ss_smem, *s_x = s_dt + SS_CHUNK * SS_CHANNELS, *s_y = s_x + SS_CHUNK * SS_CHANNELS;      // s_y: [chunk][threads]
    float *s_B = s_y + SS_CHUNK * SS_THREADS, *s_C = s_B + SS_CHUNK * a.N;
    const int req = blockIdx.y;
    const int part = threadIdx.x % SS_LANES, cl = threadIdx.x / SS_LANES;
    const int c0 = blockIdx.x * SS_CHANNELS, c = c0 + cl;
    const bool live = c < a.E;
    const int cc = live ? c : a.E - 1;          // idle lanes follow a real channel so that the shuffles stay whole
    const int first = a.req_start[req], last = a.req_start[req + 1];
    float *S = a.state + ((size_t)a.slot_ids[req] * a.E + cc) * a.N;
    float s[NPER], An[NPER];
#pragma unroll
    for (int i = 0; i < NPER; ++i) {
        const int n = part + SS_LANES * i;
        s[i] = n < a.N ? S[n] : 0.f;
        An[i] = n < a.N ? a.A[(size_t)cc * a.N + n] : 0.f;
    }
    for (int t0 = first; t0 < last; t0 += SS_CHUNK) {
        const int n_rows = min(SS_CHUNK, last - t0);
        // the loops below are unrolled so that a thread's loads are asked for together, not one after the other's arrival
#pragma unroll 4
        for (int idx = threadIdx.x; idx < SS_CHUNK * SS_CHANNELS; idx += SS_THREADS) {
            const int tt = idx / SS_CHANNELS, ch = min(c0 + idx % SS_CHANNELS, a.E - 1);
            if (tt >= n_rows) { s_dt[idx] = 0.f; s_x[idx] = 0.f; continue; }
            const size_t t = (size_t)(t0 + tt);
            float dt;
            if (a.dt != nullptr) {
                dt = a.dt[t * a.ld_dt + ch];
            } else {
                const float *low = a.low + t * a.ld_low;
                const T *w = (const T *)a.Wdt + (size_t)ch * a.K;
                float d = 0.f;
                for (int k = 0; k < a.K; ++k) d = fmaf(to_f32(w[k]), low[k], d);
                dt = softplus_f(d + a.bdt[ch]);
            }
            s_dt[idx] = dt;
            s_x[idx] = a.x[t * a.E + ch];
        }
#pragma unroll 4
        for (int idx = threadIdx.x; idx < SS_CHUNK * a.N; idx += SS_THREADS) {
            const int tt = idx / a.N, n = idx % a.N;
            const float *low = a.low + (size_t)(t0 + min(tt, n_rows - 1)) * a.ld_low + a.K;
            s_B[idx] = low[n];
            s_C[idx] = low[a.N + n];
        }
        __syncthreads();
        // four rows at a time: their step sizes, inputs, B and C into registers first, then the four updates in order, then
        // the four shares; rows beyond the chunk's end were staged as dt = 0, x = 0 and leave the state as it is
        for (int t4 = 0; t4 < n_rows; t4 += 4) {
            float dt4[4], dx4[4], B4[4][NPER], C4[4][NPER], y4[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                dt4[j] = s_dt[(t4 + j) * SS_CHANNELS + cl];
                dx4[j] = dt4[j] * s_x[(t4 + j) * SS_CHANNELS + cl];
#pragma unroll
                for (int i = 0; i < NPER; ++i) {
                    const int n = part + SS_LANES * i;
                    B4[j][i] = n < a.N ? s_B[(t4 + j) * a.N + n] : 0.f;
                    C4[j][i] = n < a.N ? s_C[(t4 + j) * a.N + n] : 0.f;
                }
            }
            float decay[4][NPER];
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int i = 0; i < NPER; ++i) decay[j][i] = expf(dt4[j] * An[i]);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float y = 0.f;
#pragma unroll
                for (int i = 0; i < NPER; ++i) {
                    s[i] = fmaf(decay[j][i], s[i], dx4[j] * B4[j][i]);
                    y = fmaf(s[i], C4[j][i], y);
                }
                y4[j] = y;
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) s_y[(t4 + j) * SS_THREADS + threadIdx.x] = y4[j];
        }
        __syncthreads();
#pragma unroll 4
        for (int idx = threadIdx.x; idx < n_rows * SS_CHANNELS; idx += SS_THREADS) {
            const int tt = idx / SS_CHANNELS, k = idx % SS_CHANNELS, ch = c0 + k;
            if (ch < a.E) {
                const size_t t = (size_t)(t0 + tt);
                const float *share = s_y + tt * SS_THREADS + k * SS_LANES;
                float y = 0.f;
#pragma unroll
                for (int i = 0; i < SS_LANES; ++i) y += share[i];
                y = fmaf(a.Dskip[ch], s_x[idx], y);
                ((T *)a.out)[t * a.E + ch] = from_f32<T>(y * silu_f(a.z[t * a.ld_z + ch]));
            }
        }
        __syncthreads();        // the next chunk's rows overwrite what this pass still reads
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < NPER; ++i) {
            const int n = part + SS_LANES * i;
            if (n < a.N) S[n] = s[i];
        }
    }
}

// `dt_buf` (may be null): room for step sizes [T, ld_dt], made ahead with one product; without it they are formed while
// the rows are staged.  `Wdt` is of the type `dtype` names.
JK_EXPORT int jk_selective_scan(const float *x, const float *low, int ld_low, int K, int N, int E, const float *z, int ld_z,
                                const void *Wdt, const float *bdt, const float *A, const float *Dskip, float *state,
                                const int *req_start, const int *slot_ids, int nreq, void *out, int dtype, float *dt_buf, int ld_dt,
                                int T, cudaStream_t stream) {
    if (nreq == 0) return JK_OK;
    JK_REQUIRE(x && low && z && Wdt && bdt && A && Dskip && state && req_start && slot_ids && out, "selective_scan: an argument is missing");
    JK_REQUIRE(K > 0 && N > 0 && E > 0 && ld_low >= K + 2 * N, "selective_scan: rank %d, states %d, channels %d, rows of %d", K, N, E, ld_low);
    JK_REQUIRE(N <= SS_LANES * 32, "selective_scan: %d states exceed %d", N, SS_LANES * 32);
    JK_REQUIRE(nreq <= 65535, "selective_scan: %d requests exceed one launch", nreq);
    const bool ahead = dt_buf != nullptr;
    if (ahead) {
        const dim3 tiles((T + GT_M - 1) / GT_M, (E + GT_N - 1) / GT_N);
#define LAUNCH(TT) jk_launch(scan_steps_kernel<TT>, tiles, dim3(256), 0, stream, low, ld_low, (const TT *)Wdt, bdt, dt_buf, ld_dt, T, E, K)
        BLOCKS_BY_DTYPE(dtype, "scan_steps", LAUNCH);
#undef LAUNCH
        JK_CHECK_LAUNCH("scan_steps");
    }
    ScanArgs a{x, low, ld_low, K, N, E, z, ld_z, Wdt, bdt, A, Dskip, state, req_start, slot_ids, out, ahead ? dt_buf : nullptr, ld_dt};
    dim3 grid((E + SS_CHANNELS - 1) / SS_CHANNELS, nreq);
    const int per = (N + SS_LANES - 1) / SS_LANES;
    const size_t smem = (size_t)SS_CHUNK * (2 * SS_CHANNELS + SS_THREADS + 2 * N) * sizeof(float);
#define LAUNCH_N(TT, NPER)                                                                                                                  \
    do {                                                                                                                                    \
        if (smem > 46 * 1024) cudaFuncSetAttribute(selective_scan_kernel<TT, NPER>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        jk_launch(selective_scan_kernel<TT, NPER>, grid, dim3(SS_THREADS), smem, stream, a);                                                \
    } while (0)
#define LAUNCH(TT)                              \
    if (per <= 1) LAUNCH_N(TT, 1);              \
    else if (per <= 2) LAUNCH_N(TT, 2);         \
    else if (per <= 4) LAUNCH_N(TT, 4);         \
    else if (per <= 8) LAUNCH_N(TT, 8);         \
    else if (per <= 16) LAUNCH_N(TT, 16);       \
    else LAUNCH_N(TT, 32)
    BLOCKS_BY_DTYPE(dtype, "selective_scan", LAUNCH);
#undef LAUNCH
#undef LAUNCH_N
    JK_CHECK_LAUNCH("selective_scan");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// Routed experts.  route_topk: a block per row or per four rows; logits z_e = router[e] . h in float32, scores sigmoid(z_e); the `top`
// experts of largest score (the lower index wins a tie) -> ids, scores [T, top], and the experts' counts.  route_sort:
// one block per expert lists its (row, choice) pairs in the order of the rows: entry -> source row, score; pair -> entry.
// The experts' products then run over the entries, expert after expert, as tiles of the grouped kernels below; an
// expert's input is score * h, which the first product applies to its sums (W (s h) = s (W h), in float32) before the
// gate's activation.  expert_combine adds a row's `top` results in the order of its choices.
// Options: a bias on the logits (`bias` [E]); a gate per row, sigmoid(gate_w . h), on what the sum is added to (a shared
// unit's output that waits in delta).
// ---------------------------------------------------------------------------------------------------------------
template <typename T> struct Vec16;
template <> struct Vec16<float> { static constexpr int N = 4; };
template <> struct Vec16<__nv_bfloat16> { static constexpr int N = 8; };

template <typename T>
__device__ __forceinline__ void unpack16(const uint4 &v, float *f) {
    if constexpr (Vec16<T>::N == 4) {
        f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y); f[2] = __uint_as_float(v.z); f[3] = __uint_as_float(v.w);
    } else {
        const unsigned w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(w[i] << 16); f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
    }
}

// eight elements of a row that starts on a 16-byte boundary
__device__ __forceinline__ void load8(const float *p, float *f) {
    *reinterpret_cast<float4 *>(f) = *reinterpret_cast<const float4 *>(p);
    *reinterpret_cast<float4 *>(f + 4) = *reinterpret_cast<const float4 *>(p + 4);
}
__device__ __forceinline__ void load8(const __nv_bfloat16 *p, float *f) { unpack16<__nv_bfloat16>(*reinterpret_cast<const uint4 *>(p), f); }

// The largest of n values (the lower index wins a tie) over a warp; every lane gets (value, index).  An index within the
// list whatever the values are.
__device__ __forceinline__ int warp_argmax(const float *v, int n, float *value) {
    const int lane = threadIdx.x & 31;
    float best = -INFINITY;
    int at = n;
    for (int e = lane; e < n; e += 32)
        if (v[e] > best) { best = v[e]; at = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int oa = __shfl_xor_sync(0xffffffffu, at, o);
        if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
    }
    *value = best;
    return at < n ? at : n - 1;
}

// N router outputs, of which the first E stand for experts with matrices and the rest for units that return their input.
// score_form 0: sigmoid; 1: softmax over all, the chosen ones' scores divided by their sum, times score_scale; 2: softmax over all, as they are.
// Forms 0 and 1 choose by the logits, form 2 by score + correction; with groups only outputs of the `group_keep` groups
// (of N / group_count neighbours) whose best choice score is largest can be chosen.  A block takes R rows: a warp one output
// at a time for all of them (a router row is read once a block), then a warp a row for the choice.
struct RouteArgs {
    const float *router, *bias, *gate_w, *correction;
    int T, D, N, E, top, score_form, group_count, group_keep;
    int *ids, *counts;
    float *scores, *row_gate;
    float score_scale;          // form 1: factor of the renormalised scores
};

template <typename T, int R>
__global__ void route_topk_kernel(const T *__restrict__ h, RouteArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float route_smem[];       // per row: [N] logits, then scores; [N] choice scores; [group_count] best of a group, kept
    const int N = a.N, D = a.D, row_floats = 2 * N + 2 * a.group_count;
    const int t0 = blockIdx.x * R, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
    const bool vec = D % 8 == 0 && (uintptr_t)h % 16 == 0 && (uintptr_t)a.router % 16 == 0 && (uintptr_t)a.gate_w % 16 == 0;
    // output N: the row's gate on what the experts' sum is added to
    for (int e = warp; e < (a.gate_w != nullptr ? N + 1 : N); e += nwarp) {
        const float *w = e < N ? a.router + (size_t)e * D : a.gate_w;
        float dot[R];
#pragma unroll
        for (int r = 0; r < R; ++r) dot[r] = 0.f;
        if (vec) {          // eight elements a lane a pass, the passes' loads independent of one another
#pragma unroll 4
            for (int c = lane * 8; c < D; c += 256) {
                float wv[8];
                load8(w + c, wv);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    float x[8];
                    load8(h + (size_t)min(t0 + r, a.T - 1) * D + c, x);
#pragma unroll
                    for (int i = 0; i < 8; ++i) dot[r] = fmaf(wv[i], x[i], dot[r]);
                }
            }
        } else {
            for (int c = lane; c < D; c += 32)
#pragma unroll
                for (int r = 0; r < R; ++r) dot[r] = fmaf(w[c], to_f32(h[(size_t)min(t0 + r, a.T - 1) * D + c]), dot[r]);
        }
#pragma unroll
        for (int r = 0; r < R; ++r) {
            dot[r] = warp_sum(dot[r]);
            if (lane != 0) continue;
            if (e < N) route_smem[r * row_floats + e] = dot[r] + (a.bias ? a.bias[e] : 0.f);
            else if (t0 + r < a.T) a.row_gate[t0 + r] = sigmoid_f(dot[r]);
        }
    }
    __syncthreads();
    const int t = t0 + warp;
    if (warp >= R || t >= a.T) return;
    float *z = route_smem + warp * row_floats, *choice = z + N, *group_best = choice + N, *group_kept = group_best + a.group_count;
    float zmax = -INFINITY, total = 0.f, unused;
    if (a.score_form != 0) {
        for (int e = lane; e < N; e += 32) zmax = fmaxf(zmax, z[e]);
        zmax = warp_max(zmax);
        for (int e = lane; e < N; e += 32) total += expf(z[e] - zmax);
        total = warp_sum(total);
    }
    for (int e = lane; e < N; e += 32) {        // a lane's own outputs: no other lane touches them before the barrier
        const float logit = z[e], s = a.score_form != 0 ? expf(logit - zmax) / total : sigmoid_f(logit);
        choice[e] = a.score_form == 2 ? s + (a.correction ? a.correction[e] : 0.f) : logit;
        z[e] = s;
    }
    __syncwarp();
    if (a.group_count > 0) {
        const int size = N / a.group_count;
        for (int g = lane; g < a.group_count; g += 32) {
            float b = -INFINITY;
            for (int i = 0; i < size; ++i) b = fmaxf(b, choice[g * size + i]);
            group_best[g] = b;
            group_kept[g] = 0.f;
        }
        __syncwarp();
        for (int k = 0; k < a.group_keep; ++k) {
            const int g = warp_argmax(group_best, a.group_count, &unused);
            __syncwarp();
            if (lane == 0) { group_best[g] = -INFINITY; group_kept[g] = 1.f; }
            __syncwarp();
        }
        for (int e = lane; e < N; e += 32)
            if (group_kept[e / size] == 0.f) choice[e] = -INFINITY;
        __syncwarp();
    }
    float chosen = 0.f;
    int *ids = a.ids + (size_t)t * a.top;
    float *scores = a.scores + (size_t)t * a.top;
    for (int k = 0; k < a.top; ++k) {
        const int best = warp_argmax(choice, N, &unused);
        const float sc = z[best];
        chosen += sc;
        __syncwarp();
        if (lane == 0) {
            ids[k] = best;
            scores[k] = sc;
            if (best < a.E) atomicAdd(&a.counts[best], 1);
            choice[best] = -INFINITY;
        }
        __syncwarp();
    }
    if (a.score_form == 1)
        for (int k = lane; k < a.top; k += 32) scores[k] = scores[k] / (chosen + 1e-20f) * a.score_scale;
}

// entry_row[pos], entry_score[pos] for pos in [starts[e], starts[e + 1]); pair_entry[pair] = pos.  A block an expert; each of its
// warps takes a stretch of the pairs: it counts the expert's among them, and behind the barrier lists them from where the
// warps before it end, so the entries are in the order of the rows.
constexpr int RS_WARPS = 32;

__global__ void route_sort_kernel(const int *__restrict__ ids, const float *__restrict__ scores, const int *__restrict__ counts, int pairs,
                                  int E, int top, int *__restrict__ starts, int *__restrict__ entry_row, float *__restrict__ entry_score,
                                  int *__restrict__ pair_entry) {
    pdl_trigger();
    pdl_wait();
    __shared__ int found[RS_WARPS];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5, e = blockIdx.x;
    int start = 0;
    for (int i = lane; i < e; i += 32) start += counts[i];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) start += __shfl_xor_sync(0xffffffffu, start, o);
    if (threadIdx.x == 0) {
        starts[e] = start;
        if (e == E - 1) starts[E] = start + counts[e];
    }
    const int stretch = ((pairs + nwarp - 1) / nwarp + 31) / 32 * 32, first = warp * stretch, end = min(pairs, first + stretch);
    int mine = 0;
#pragma unroll 4
    for (int p = first + lane; p < end; p += 32) mine += ids[p] == e ? 1 : 0;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mine += __shfl_xor_sync(0xffffffffu, mine, o);
    if (lane == 0) found[warp] = mine;
    __syncthreads();
    int at = start;
    for (int i = 0; i < warp; ++i) at += found[i];
    if (mine == 0) return;
    for (int p0 = first; p0 < end; p0 += 32) {
        const int p = p0 + lane;
        const bool hit = p < end && ids[p] == e;
        const unsigned ballot = __ballot_sync(0xffffffffu, hit);
        if (hit) {
            const int pos = at + __popc(ballot & ((1u << lane) - 1u));
            entry_row[pos] = p / top;
            entry_score[pos] = scores[p];
            pair_entry[p] = pos;
        }
        at += __popc(ballot);
    }
}

// which expert's tile a block has: tiles of GT_M entries, expert after expert
__device__ __forceinline__ bool expert_tile(const int *starts, int E, int block, int *expert, int *m0) {
    int tiles = 0;
    for (int e = 0; e < E; ++e) {
        const int n = starts[e + 1] - starts[e];
        const int mine = (n + GT_M - 1) / GT_M;
        if (block < tiles + mine) { *expert = e; *m0 = (block - tiles) * GT_M; return true; }
        tiles += mine;
    }
    return false;
}

// act[entry, n] = T(actf(s * g) * (s * u)), g = W_gate[e] h_row, u = W_up[e] h_row; w: [E, 2 ff, D] (gate rows, then up rows)
template <typename T>
__global__ void __launch_bounds__(256) expert_gate_up_kernel(const T *__restrict__ h, const T *__restrict__ w, T *__restrict__ act, int D, int ff, int E,
                                                             const int *__restrict__ starts, const int *__restrict__ entry_row,
                                                             const float *__restrict__ entry_score, int actf, float limit) {
    pdl_trigger();
    pdl_wait();
    int e, m0;
    if (!expert_tile(starts, E, blockIdx.x, &e, &m0)) return;
    const int first = starts[e], M = starts[e + 1] - first, n0 = blockIdx.y * GT_N;
    const T *we = w + (size_t)e * 2 * ff * D;
    float g[16], u[16];
    tile_product<true>(h, (size_t)D, entry_row + first, M, we, we + (size_t)ff * D, (size_t)D, ff, D, m0, n0, g, u);
#pragma unroll
    for (int e = 0; e < 16; ++e) {
        int r, c;
        tile_at<T>(e, &r, &c);
        r += m0;
        const int n = n0 + c;
        if (r >= M || n >= ff) continue;
        const float s = entry_score ? entry_score[first + r] : 1.f;
        act[(size_t)(first + r) * ff + n] = from_f32<T>(expert_inner(actf, s, g[e], u[e], limit));
    }
}

// y[entry, n] = W_down[e] act[entry]; w: [E, D, ff]; float32 out
template <typename T>
__global__ void __launch_bounds__(256) expert_down_kernel(const T *__restrict__ act, const T *__restrict__ w, float *__restrict__ y, int D, int ff, int E,
                                                          const int *__restrict__ starts) {
    pdl_trigger();
    pdl_wait();
    int e, m0;
    if (!expert_tile(starts, E, blockIdx.x, &e, &m0)) return;
    const int first = starts[e], M = starts[e + 1] - first, n0 = blockIdx.y * GT_N;
    float acc[16], unused[16];
    tile_product<false>(act + (size_t)first * ff, (size_t)ff, nullptr, M, w + (size_t)e * D * ff, (const T *)nullptr, (size_t)ff, D, ff, m0, n0, acc, unused);
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        int r, c;
        tile_at<T>(i, &r, &c);
        r += m0;
        const int n = n0 + c;
        if (r < M && n < D) y[(size_t)(first + r) * D + n] = acc[i];
    }
}

// Steps of few rows (decoding): an expert has a handful of entries, and its matrices only have to stream past them.  A
// block of eight warps takes one expert and a slice of its output features; the expert's entries (up to ER_ROWS at a
// time) wait in shared memory; a warp takes one feature at a time, its lanes 16 bytes of the weight row each
// per pass, all loads of a row asked for before the sums start.  Float32 sums on the CUDA cores, in the order of K per
// lane and then across lanes, whatever else the step holds.
constexpr int ER_ROWS = 8, ER_FEATURES = 32;        // entries at a time; output features a block

// the features of one block against ROWS staged entries (the caller picks the smallest ROWS that holds them)
template <typename T, bool GLU, int ROWS>
__device__ __forceinline__ void expert_rows_features(const T *__restrict__ er_rows, const T *__restrict__ we, void *__restrict__ out, int K, int N,
                                                     int rows, size_t entry0, const float *__restrict__ entry_score, int actf, float limit) {
    constexpr int V = Vec16<T>::N;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int f = warp; f < ER_FEATURES; f += 8) {
        const int n = blockIdx.y * ER_FEATURES + f;
        if (n >= N) break;
        const T *wg = we + (size_t)n * K, *wu = we + (size_t)(N + n) * K;
        float g[ROWS], u[ROWS];
#pragma unroll
        for (int r = 0; r < ROWS; ++r) { g[r] = 0.f; u[r] = 0.f; }
#pragma unroll 4
        for (int k = lane * V; k < K; k += 32 * V) {
            float a[V], b[V];
            unpack16<T>(*reinterpret_cast<const uint4 *>(wg + k), a);
            if (GLU) unpack16<T>(*reinterpret_cast<const uint4 *>(wu + k), b);
#pragma unroll
            for (int r = 0; r < ROWS; ++r) {
                float x[V];
                unpack16<T>(*reinterpret_cast<const uint4 *>(er_rows + r * K + k), x);
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    g[r] = fmaf(a[i], x[i], g[r]);
                    if (GLU) u[r] = fmaf(b[i], x[i], u[r]);
                }
            }
        }
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            g[r] = warp_sum(g[r]);
            if (GLU) u[r] = warp_sum(u[r]);
        }
        if (lane == 0) {
#pragma unroll
            for (int r = 0; r < ROWS; ++r) {
                if (r >= rows) break;
                const size_t entry = entry0 + r;
                if (GLU) {
                    const float sc = entry_score ? entry_score[entry] : 1.f;
                    ((T *)out)[entry * N + n] = from_f32<T>(expert_inner(actf, sc, g[r], u[r], limit));
                } else {
                    ((float *)out)[entry * N + n] = g[r];
                }
            }
        }
    }
}

// GLU: act[entry, n] = T(actf(s g) (s u)) from rows of h picked by entry_row; else y[entry, n] = W[e][n] . in[entry]
template <typename T, bool GLU>
__global__ void __launch_bounds__(256) expert_rows_kernel(const T *__restrict__ in, const T *__restrict__ w, void *__restrict__ out, int K, int N, int E,
                                                          const int *__restrict__ starts, const int *__restrict__ entry_row,
                                                          const float *__restrict__ entry_score, int actf, float limit) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char er_smem[];
    T *er_rows = reinterpret_cast<T *>(er_smem);             // [ER_ROWS][K] as they are stored
    const int e = blockIdx.x, first = starts[e], M = starts[e + 1] - first;
    if (M <= 0) return;
    constexpr int V = Vec16<T>::N;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const T *we = w + (size_t)e * (GLU ? 2 : 1) * N * K;
    for (int r0 = 0; r0 < M; r0 += ER_ROWS) {
        const int rows = min(ER_ROWS, M - r0);
        __syncthreads();
        if (warp < rows) {      // warp r brings entry r: one look at where it lies, then 16 bytes a lane a pass
            const T *src = in + (size_t)(GLU ? entry_row[first + r0 + warp] : first + r0 + warp) * K;
#pragma unroll 4
            for (int k = lane * V; k < K; k += 32 * V)
                *reinterpret_cast<uint4 *>(er_rows + warp * K + k) = *reinterpret_cast<const uint4 *>(src + k);
        }
        __syncthreads();
        const size_t entry0 = (size_t)(first + r0);
        if (rows <= 1) expert_rows_features<T, GLU, 1>(er_rows, we, out, K, N, rows, entry0, entry_score, actf, limit);
        else if (rows <= 2) expert_rows_features<T, GLU, 2>(er_rows, we, out, K, N, rows, entry0, entry_score, actf, limit);
        else if (rows <= 4) expert_rows_features<T, GLU, 4>(er_rows, we, out, K, N, rows, entry0, entry_score, actf, limit);
        else expert_rows_features<T, GLU, 8>(er_rows, we, out, K, N, rows, entry0, entry_score, actf, limit);
    }
}

// v[t] = (what waits in delta, times the row's gate, if `add`) + sum over the row's choices, in their order, of y[pair_entry[t *
// top + k]], times the choice's score where scores multiply a unit's output (`out_scores`); a choice beyond the E experts is
// the row's own input h[t].  delta[t] = v, or with a stream x: x[t] += x_scale * v + pend_scale * pend[t] (a product that waits
// for the stream).  V elements a thread.
struct CombineArgs {
    const float *y;
    const int *pair_entry, *ids;
    const float *out_scores;        // [T, top] or null
    int E, D, top, add;
    float *delta;
    const float *row_gate;
    const void *h;
    float *x;
    float x_scale;
    const float *pend;
    float pend_scale;
};

template <typename T, int V>
__global__ void expert_combine_kernel(CombineArgs a, size_t total) {
    pdl_trigger();
    pdl_wait();
    struct __align__(4 * V) Vec { float f[V]; };
    struct __align__(sizeof(T) * V) VecT { T f[V]; };
    for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V; i < total; i += (size_t)gridDim.x * blockDim.x * V) {
        const size_t t = i / a.D;
        const int c = (int)(i % a.D);
        Vec v;
        if (a.add) {
            v = *reinterpret_cast<const Vec *>(a.delta + i);
            if (a.row_gate) {
                const float g = a.row_gate[t];
#pragma unroll
                for (int e = 0; e < V; ++e) v.f[e] *= g;
            }
        } else {
#pragma unroll
            for (int e = 0; e < V; ++e) v.f[e] = 0.f;
        }
        for (int k = 0; k < a.top; ++k) {
            const size_t pair = t * a.top + k;
            const float s = a.out_scores ? a.out_scores[pair] : 1.f;
            if (a.ids[pair] < a.E) {
                const Vec u = *reinterpret_cast<const Vec *>(a.y + (size_t)a.pair_entry[pair] * a.D + c);
#pragma unroll
                for (int e = 0; e < V; ++e) v.f[e] = fmaf(s, u.f[e], v.f[e]);
            } else {
                const VecT u = *reinterpret_cast<const VecT *>((const T *)a.h + i);
#pragma unroll
                for (int e = 0; e < V; ++e) v.f[e] = fmaf(s, to_f32(u.f[e]), v.f[e]);
            }
        }
        if (a.x != nullptr) {
            Vec x = *reinterpret_cast<const Vec *>(a.x + i);
            if (a.pend != nullptr) {
                const Vec p = *reinterpret_cast<const Vec *>(a.pend + i);
#pragma unroll
                for (int e = 0; e < V; ++e) x.f[e] = fmaf(a.pend_scale, p.f[e], x.f[e]);
            }
#pragma unroll
            for (int e = 0; e < V; ++e) x.f[e] = fmaf(a.x_scale, v.f[e], x.f[e]);
            *reinterpret_cast<Vec *>(a.x + i) = x;
        } else {
            *reinterpret_cast<Vec *>(a.delta + i) = v;
        }
    }
}

// ints of workspace (`route`) that T rows need: counts [N], starts [N + 1], ids, entry_row, pair_entry [T top] and, as
// floats, scores and entry_score [T top] and the rows' gates [T]; N counts the router's outputs
JK_EXPORT long long jk_routed_experts_workspace(int T, int N, int top) { return 2LL * N + 1 + 5LL * T * top + T + 16; }

// h [T, D] (type T) -> delta [T, D] float32 (add: on top of what is there), or into the stream x (x += x_scale * sum + pend_scale
// * pend).  entries [T top, D]-sized buffers: `act` [T top, ff] of the activation type, `y` [T top, D] float32.
// router [E + identity, D]; group_count 0: no groups.
JK_EXPORT int jk_routed_experts(const void *h, const float *router, const void *w_gate_up, const void *w_down, float *delta, int add,
                                int dtype, int T, int D, int ff, int E, int top, int actf, int *route, void *act, float *y,
                                int score_form, float limit, const float *router_bias, const float *gate_w, int identity, int group_count,
                                int group_keep, const float *correction, float *x, float x_scale, const float *pend, float pend_scale,
                                float score_scale, cudaStream_t stream) {
    if (T == 0) return JK_OK;
    const int N = E + identity;
    JK_REQUIRE(gate_w == nullptr || add, "routed_experts: a gate on a shared unit's output that is not there");
    JK_REQUIRE(h && router && w_gate_up && w_down && delta && route && act && y, "routed_experts: an argument is missing");
    JK_REQUIRE(D > 0 && ff > 0 && E > 0 && identity >= 0 && top > 0 && top <= N, "routed_experts: %d + %d experts, %d a row, sizes %d and %d", E, identity, top, D, ff);
    JK_REQUIRE(score_form >= 0 && score_form <= 2 && (identity == 0 || score_form != 0), "routed_experts: scores of form %d with %d identities", score_form, identity);
    JK_REQUIRE(correction == nullptr || score_form == 2, "routed_experts: a correction of the choice with scores of form %d", score_form);
    JK_REQUIRE(group_count == 0 || (group_count > 0 && N % group_count == 0 && group_keep > 0 && group_keep <= group_count && group_keep * (N / group_count) >= top),
               "routed_experts: %d of %d groups of %d outputs for %d choices", group_keep, group_count, N, top);
    JK_REQUIRE(pend == nullptr || x != nullptr, "routed_experts: a product that waits needs the stream");
    JK_REQUIRE(score_scale == 1.f || score_form == 1, "routed_experts: a factor of scores of form %d", score_form);
    const size_t route_smem = (2 * (size_t)N + 2 * (size_t)group_count) * sizeof(float);
    JK_REQUIRE(route_smem <= 40 * 1024, "routed_experts: %d experts exceed the router's shared memory", N);
    const int pairs = T * top;
    int *counts = route, *starts = counts + E, *ids = starts + E + 1, *entry_row = ids + pairs, *pair_entry = entry_row + pairs;
    float *scores = (float *)(pair_entry + pairs), *entry_score = scores + pairs, *row_gate = gate_w ? entry_score + pairs : nullptr;
    if (cudaMemsetAsync(counts, 0, sizeof(int) * (size_t)E, stream) != cudaSuccess) JK_FAIL(JK_CUDA_ERROR, "routed_experts: clearing the counts failed");
    const RouteArgs ra{router, router_bias, gate_w, correction, T, D, N, E, top, score_form, group_count, group_keep, ids, counts, scores, row_gate, score_scale};
    // few rows: a block a row with a warp for every output; many: four rows a block
    const int many = T >= 512 && 4 * route_smem <= 40 * 1024, warps = many ? 8 : std::min(32, std::max(4, N));
#define LAUNCH(TT)                                                                                                          \
    if (many) jk_launch(route_topk_kernel<TT, 4>, dim3((T + 3) / 4), dim3(32 * warps), 4 * route_smem, stream, (const TT *)h, ra); \
    else jk_launch(route_topk_kernel<TT, 1>, dim3(T), dim3(32 * warps), route_smem, stream, (const TT *)h, ra)
    BLOCKS_BY_DTYPE(dtype, "route_topk", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("route_topk");
    jk_launch(route_sort_kernel, dim3(E), dim3(32 * std::max(1, std::min(RS_WARPS, pairs / 64))), 0, stream, (const int *)ids, (const float *)scores, (const int *)counts, pairs, E, top,
              starts, entry_row, entry_score, pair_entry);
    JK_CHECK_LAUNCH("route_sort");
    // few rows: the experts' matrices stream past their entries (rows of 16-byte multiples); else tiles
    // score_form 1 and 2: the score multiplies the unit's output (in the sum of a row's choices), not its input
    const float *in_score = score_form != 0 ? nullptr : entry_score, *out_scores = score_form != 0 ? scores : nullptr;
    const int per16 = dtype == JK_F32 ? 4 : 8;
    const bool stream_rows = pairs <= 64 && D % per16 == 0 && ff % per16 == 0 && (uintptr_t)w_gate_up % 16 == 0 && (uintptr_t)w_down % 16 == 0 &&
                             (size_t)ER_ROWS * std::max(D, ff) * 4 <= 160 * 1024;
    if (stream_rows) {
        const size_t elem = dtype == JK_F32 ? 4 : 2, smem_up = (size_t)ER_ROWS * D * elem, smem_down = (size_t)ER_ROWS * ff * elem;
#define LAUNCH(TT)                                                                                                                           \
    if (smem_up > 46 * 1024) cudaFuncSetAttribute(expert_rows_kernel<TT, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_up);  \
    if (smem_down > 46 * 1024) cudaFuncSetAttribute(expert_rows_kernel<TT, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_down); \
    jk_launch(expert_rows_kernel<TT, true>, dim3(E, (ff + ER_FEATURES - 1) / ER_FEATURES), dim3(256), smem_up, stream, (const TT *)h,        \
              (const TT *)w_gate_up, act, D, ff, E, (const int *)starts, (const int *)entry_row, in_score, actf, limit);          \
    jk_launch(expert_rows_kernel<TT, false>, dim3(E, (D + ER_FEATURES - 1) / ER_FEATURES), dim3(256), smem_down, stream, (const TT *)act,    \
              (const TT *)w_down, (void *)y, ff, D, E, (const int *)starts, (const int *)nullptr, (const float *)nullptr, 0, 0.f)
        BLOCKS_BY_DTYPE(dtype, "expert rows", LAUNCH);
#undef LAUNCH
        JK_CHECK_LAUNCH("expert rows");
    } else {
    const int tiles = (pairs + GT_M - 1) / GT_M + E;
#define LAUNCH(TT)                                                                                                                          \
    jk_launch(expert_gate_up_kernel<TT>, dim3(tiles, (ff + GT_N - 1) / GT_N), dim3(256), 0, stream, (const TT *)h, (const TT *)w_gate_up,  \
              (TT *)act, D, ff, E, (const int *)starts, (const int *)entry_row, in_score, actf, limit);                          \
    jk_launch(expert_down_kernel<TT>, dim3(tiles, (D + GT_N - 1) / GT_N), dim3(256), 0, stream, (const TT *)act, (const TT *)w_down, y, D, \
              ff, E, (const int *)starts)
    BLOCKS_BY_DTYPE(dtype, "expert products", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("expert products");
    }
    const size_t total = (size_t)T * D;
    const CombineArgs ca{y, pair_entry, ids, out_scores, E, D, top, add, delta, row_gate, h, x, x_scale, pend, pend_scale};
    const bool four = D % 4 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)delta % 16 == 0 && (uintptr_t)h % 16 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)pend % 16 == 0;
    const size_t threads = total / (four ? 4 : 1);
    const int combine_blocks = (int)std::min<size_t>((threads + 255) / 256, 148 * 16);
#define LAUNCH(TT)                                                                                            \
    if (four) jk_launch(expert_combine_kernel<TT, 4>, dim3(combine_blocks), dim3(256), 0, stream, ca, total); \
    else jk_launch(expert_combine_kernel<TT, 1>, dim3(combine_blocks), dim3(256), 0, stream, ca, total)
    BLOCKS_BY_DTYPE(dtype, "expert_combine", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("expert_combine");
    return JK_OK;
}
// kernels that one call of jk_routed_experts launches (the clearing of the counts included)
JK_EXPORT int jk_routed_experts_launches() { return 6; }

// ---------------------------------------------------------------------------------------------------------------
// x[t] += table[index[t]] (index null: row `fixed` for every t): learned position vectors picked by the rows' positions,
// or one vector of a table added to the whole stream.  The table is float32 or of the compute type; the sum is float32.
// ---------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void add_rows_kernel(float *__restrict__ x, const T *__restrict__ table, const int *__restrict__ index, int fixed, int d, size_t total) {
    pdl_trigger();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / d;
        const int row = index ? index[t] : fixed;
        x[i] += to_f32(table[(size_t)row * d + (i % d)]);
    }
}

JK_EXPORT int jk_add_rows(float *x, const void *table, int table_dtype, int table_rows, const int *index, int fixed, int rows, int d,
                          cudaStream_t stream) {
    if (rows == 0) return JK_OK;
    JK_REQUIRE(x && table && d > 0 && table_rows > 0 && (index || (fixed >= 0 && fixed < table_rows)), "add_rows: row %d of a table of %d", fixed, table_rows);
    const size_t total = (size_t)rows * d;
    const int blocks = (int)std::min<size_t>((total + 255) / 256, 148 * 16);
#define LAUNCH(TT) jk_launch(add_rows_kernel<TT>, dim3(blocks), dim3(256), 0, stream, x, (const TT *)table, index, fixed, d, total)
    BLOCKS_BY_DTYPE(table_dtype, "add_rows", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("add_rows");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// logits <- cap * tanh(logits / cap)
// ---------------------------------------------------------------------------------------------------------------
__global__ void softcap_kernel(float *__restrict__ x, float cap, size_t total) {
    pdl_trigger();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) x[i] = cap * tanhf(x[i] / cap);
}

JK_EXPORT int jk_softcap(float *x, float cap, long long n, cudaStream_t stream) {
    if (n == 0) return JK_OK;
    JK_REQUIRE(x && n > 0 && cap > 0.f, "softcap: %lld values, cap %f", n, (double)cap);
    jk_launch(softcap_kernel, dim3((int)std::min<long long>((n + 255) / 256, 148 * 16)), dim3(256), 0, stream, x, cap, (size_t)n);
    JK_CHECK_LAUNCH("softcap");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// Embedding with a vector per pair of neighbouring tokens and a norm:
//     v_t = scale * table[token_t] + pairs[r_t],   r_t = (prev_t * mul_prev + token_t * mul_cur) mod buckets, or `buckets` at position 0
//     x_t = v_t / sqrt(mean(v_t^2) + eps) * w        (w null: x_t = v_t; pairs null: no second vector)
// prev_t of a portion's first row is the last token of the request's step before.  What is kept of a request is two marked tokens
// that take turns, state[slot, 2] of (positions the sequence had then, token): a step that starts at position p reads the one marked
// p and leaves its last token, marked with the new length, in the other, so the block with a request's first row and the one with
// its last never touch the same (the scheme of norm_pair's kept rows).  One block per row.
// ---------------------------------------------------------------------------------------------------------------
struct EmbedPairArgs {
    const int *tokens, *positions, *row_req, *req_start, *req_pos, *slot_ids;
    const void *table, *pairs;
    int buckets;
    long long mul_prev, mul_cur;
    float scale;
    int *state;             // [slots, 2, 2]
    const float *w;
    float eps;
    float *x;
    int d;
};

__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16 *p) {
    const uint2 v = *reinterpret_cast<const uint2 *>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}

template <typename TW, bool VEC>
__global__ void embed_pair_kernel(EmbedPairArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float row_buf[];
    __shared__ float scratch[33];
    __shared__ int pair_row;
    const int t = blockIdx.x, token = a.tokens[t];
    const TW *src = (const TW *)a.table + (size_t)token * a.d;
    if (a.pairs != nullptr && threadIdx.x == 0) {
        const int req = a.row_req[t], start = a.req_start[req], end = a.req_start[req + 1], pos = a.req_pos[req];
        int row = a.buckets;
        int *kept = nullptr;
        bool second = false;
        if (t == start || t + 1 == end) {
            kept = a.state + (size_t)a.slot_ids[req] * 4;
            second = *reinterpret_cast<volatile int *>(kept) != pos;        // the other one is marked with position pos
        }
        if (a.positions[t] > 0) {
            const int prev = t > start ? a.tokens[t - 1] : kept[second ? 3 : 1];
            row = (int)(((long long)prev * a.mul_prev + (long long)token * a.mul_cur) % a.buckets);
        }
        if (t + 1 == end) {
            int *to = kept + (second ? 0 : 2);
            to[1] = token;
            to[0] = pos + end - start;
        }
        pair_row = row;
    }
    __syncthreads();
    const TW *add = a.pairs != nullptr ? (const TW *)a.pairs + (size_t)pair_row * a.d : nullptr;
    float *dst = a.x + (size_t)t * a.d;
    float *keep = a.w == nullptr ? dst : row_buf;
    float ss = 0.f;
    if (VEC) {
        for (int c = threadIdx.x * 4; c < a.d; c += blockDim.x * 4) {
            float4 v = load4(src + c);
            v = make_float4(v.x * a.scale, v.y * a.scale, v.z * a.scale, v.w * a.scale);
            if (add != nullptr) {
                const float4 b = load4(add + c);
                v = make_float4(v.x + b.x, v.y + b.y, v.z + b.z, v.w + b.w);
            }
            *reinterpret_cast<float4 *>(keep + c) = v;
            ss += sumsq4(v);
        }
    } else {
        for (int c = threadIdx.x; c < a.d; c += blockDim.x) {
            float v = a.scale * to_f32(src[c]);
            if (add != nullptr) v += to_f32(add[c]);
            keep[c] = v;
            ss += v * v;
        }
    }
    if (a.w == nullptr) return;
    const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)a.d + a.eps);
    if (VEC) {
        for (int c = threadIdx.x * 4; c < a.d; c += blockDim.x * 4) *reinterpret_cast<float4 *>(dst + c) = scale4(load4(row_buf + c), inv, load4(a.w + c));
    } else {
        for (int c = threadIdx.x; c < a.d; c += blockDim.x) dst[c] = row_buf[c] * inv * a.w[c];
    }
}

// tables of type `dtype`; pairs [buckets + 1, d]
JK_EXPORT int jk_embed_pair(const int *tokens, const int *positions, const int *row_req, const int *req_start, const int *req_pos, const int *slot_ids,
                            const void *table, const void *pairs, int dtype, int buckets, int mul_prev, int mul_cur, float scale, int *state,
                            const float *w, float eps, float *x, int T, int d, cudaStream_t stream) {
    if (T == 0) return JK_OK;
    JK_REQUIRE(tokens && table && x && d > 0, "embed_pair: an argument is missing");
    JK_REQUIRE(pairs == nullptr || (positions && row_req && req_start && req_pos && slot_ids && state && buckets > 0 && mul_prev >= 0 && mul_cur >= 0),
               "embed_pair: a table of pairs of %d rows without the requests' last tokens", buckets);
    const size_t smem = w != nullptr ? (size_t)d * sizeof(float) : 0;
    JK_REQUIRE(smem <= 200 * 1024, "embed_pair: width %d does not fit shared memory", d);
    const EmbedPairArgs a{tokens, positions, row_req, req_start, req_pos, slot_ids, table, pairs, buckets, mul_prev, mul_cur, scale, state, w, eps, x, d};
    const bool vec = d % 4 == 0 && ((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)w | (uintptr_t)x) % 16 == 0;
    const int threads = T <= 64 ? std::min(1024, std::max(128, (d / 4 + 31) / 32 * 32)) : (d >= 2048 ? 256 : 128);
#define LAUNCH(TT)                                                                                                                     \
    do {                                                                                                                               \
        auto kernel = vec ? embed_pair_kernel<TT, true> : embed_pair_kernel<TT, false>;                                                \
        if (smem > 46 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                    \
        jk_launch(kernel, dim3(T), dim3(threads), smem, stream, a);                                                                    \
    } while (0)
    BLOCKS_BY_DTYPE(dtype, "embed_pair", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("embed_pair");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// What several sublayers side by side leave, into the stream by one kernel:
//     x[r] += f(p1[r], w1) + f(p2[r], w2) + p3[r],   f(p, w) = p / sqrt(mean(p^2) + eps) * w, or p where w is null
// (p2, p3 null: absent), and out[r] = T(x[r]) if `out` is given.  One block per row.
// ---------------------------------------------------------------------------------------------------------------
struct JoinArgs {
    float *x;
    const float *p1, *w1, *p2, *w2, *p3;
    float eps1, eps2;
    void *out;
    int d;
};

template <typename T, bool VEC>
__global__ void join_parts_kernel(JoinArgs a) {
    pdl_trigger();
    pdl_wait();
    __shared__ float scratch[64];
    constexpr int S = VEC ? 4 : 1;
    struct __align__(4 * S) Vec { float f[S]; };
    const size_t base = (size_t)blockIdx.x * a.d;
    float ss[2] = {0.f, 0.f};
    if (a.w1 != nullptr || a.w2 != nullptr) {
        for (int c = threadIdx.x * S; c < a.d; c += blockDim.x * S) {
            const Vec v = *reinterpret_cast<const Vec *>(a.p1 + base + c);
#pragma unroll
            for (int e = 0; e < S; ++e) ss[0] += v.f[e] * v.f[e];
            if (a.p2 != nullptr) {
                const Vec u = *reinterpret_cast<const Vec *>(a.p2 + base + c);
#pragma unroll
                for (int e = 0; e < S; ++e) ss[1] += u.f[e] * u.f[e];
            }
        }
        block_sums<2>(ss, scratch);
    }
    const float inv1 = a.w1 != nullptr ? 1.f / sqrtf(ss[0] / (float)a.d + a.eps1) : 1.f;
    const float inv2 = a.w2 != nullptr ? 1.f / sqrtf(ss[1] / (float)a.d + a.eps2) : 1.f;
    for (int c = threadIdx.x * S; c < a.d; c += blockDim.x * S) {        // the row again: it comes from the caches
        Vec x = *reinterpret_cast<const Vec *>(a.x + base + c), v = *reinterpret_cast<const Vec *>(a.p1 + base + c), w;
        if (a.w1 != nullptr) {
            w = *reinterpret_cast<const Vec *>(a.w1 + c);
#pragma unroll
            for (int e = 0; e < S; ++e) v.f[e] *= inv1 * w.f[e];
        }
        if (a.p2 != nullptr) {
            const Vec u = *reinterpret_cast<const Vec *>(a.p2 + base + c);
            if (a.w2 != nullptr) w = *reinterpret_cast<const Vec *>(a.w2 + c);
#pragma unroll
            for (int e = 0; e < S; ++e) v.f[e] += a.w2 != nullptr ? u.f[e] * inv2 * w.f[e] : u.f[e];
        }
        if (a.p3 != nullptr) {
            const Vec u = *reinterpret_cast<const Vec *>(a.p3 + base + c);
#pragma unroll
            for (int e = 0; e < S; ++e) v.f[e] += u.f[e];
        }
#pragma unroll
        for (int e = 0; e < S; ++e) x.f[e] += v.f[e];
        *reinterpret_cast<Vec *>(a.x + base + c) = x;
        if (a.out != nullptr) {
            if constexpr (VEC) store4((T *)a.out + base + c, make_float4(x.f[0], x.f[1], x.f[2], x.f[3]));
            else ((T *)a.out)[base + c] = from_f32<T>(x.f[0]);
        }
    }
}

JK_EXPORT int jk_join_parts(float *x, const float *p1, const float *w1, float eps1, const float *p2, const float *w2, float eps2, const float *p3,
                            void *out, int dtype, int rows, int d, cudaStream_t stream) {
    if (rows == 0) return JK_OK;
    JK_REQUIRE(x && p1 && rows > 0 && d > 0 && (w2 == nullptr || p2 != nullptr), "join_parts: an argument is missing");
    const bool vec = d % 4 == 0 && ((uintptr_t)x | (uintptr_t)p1 | (uintptr_t)w1 | (uintptr_t)p2 | (uintptr_t)w2 | (uintptr_t)p3 | (uintptr_t)out) % 16 == 0;
    const JoinArgs a{x, p1, w1, p2, w2, p3, eps1, eps2, out, d};
    int threads = d >= 4096 ? 512 : (d >= 1024 ? 256 : 128);
    if (rows <= 64 && vec) threads = std::min(1024, std::max(threads, (d / 4 + 31) / 32 * 32));
#define LAUNCH(T)                                                                                      \
    if (vec) jk_launch(join_parts_kernel<T, true>, dim3(rows), dim3(threads), 0, stream, a);           \
    else jk_launch(join_parts_kernel<T, false>, dim3(rows), dim3(threads), 0, stream, a)
    BLOCKS_BY_DTYPE(dtype, "join_parts", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("join_parts");
    return JK_OK;
}

// ---------------------------------------------------------------------------------------------------------------
// A real-gated linear recurrence, per channel c of C over a request's rows in order:
//     r = sigmoid(R u_t + rb)[c],  i = sigmoid(I u_t + ib)[c],  log a = rate[c] r,  a = exp(log a)
//     S <- a S + sqrt(1 - a^2) i u_t[c];      out_t[c] = T(S * act(y_t[c] + yb[c]))
// u float32 [T, C].  R and I are block-diagonal: C is cut into `blocks` equal parts of n channels, each with its own n x n matrices
// (w_r, w_i [blocks, n, n], rows are outputs); rate[c] is negative (so a < 1), and y is a column range of float32 rows.  The state
// S lives in state[slot, c], float32.  Everything is float32; in bfloat16 mode the float32 rows u meet the stored weights on the
// tensor cores as two bfloat16 halves each, so that nothing of them is rounded away.
//
// Three ways:
//   every request brings one row      gated_rows: gates, state and output of 8 rows x 16 channels a block
//   else                              gated_pairs makes (a, sqrt(1 - a^2) i u) of every row as one tiled product per part;
//                                     gated_scan then walks the work items: a request of at most SCAN_PIECE rows from its slot and
//                                     back; of a longer one, cut into pieces, the first piece from the slot (its rows leave at
//                                     once), the others from zeros (leaving their end state and the product of their decays);
//                                     gated_finish gives the other pieces their start state, the pieces before them joined in
//                                     order, and walks them again; the last one leaves the slot.  Nothing is divided by a decay.
// ---------------------------------------------------------------------------------------------------------------
struct GatedArgs {
    const float *u;
    const void *w_r, *w_i;
    const float *b_r, *b_i, *rate;
    const float *y;             // y_t[c] = y[t * ld_y + c]
    int ld_y;
    const float *y_bias;
    int act;
    float *state;
    const int *req_start, *slot_ids;
    void *out;                  // [T, C]
    int T, C, blocks, n;
    float *a, *b;               // [T, C] each: the recurrence's pairs
    float *piece_end, *piece_prod;      // [n_pieces, C]
    const int *direct, *pieces, *piece_reqs;
    int n_direct, n_pieces, n_piece_reqs;
};

// (a, sqrt(1 - a^2) i u) from the two gates' sums
__device__ __forceinline__ void gated_pair(float zr, float zi, float rate, float u, float *a, float *b) {
    const float la = rate * sigmoid_f(zr);
    *a = expf(la);
    *b = sqrtf(-expm1f(2.f * la)) * sigmoid_f(zi) * u;
}

template <typename TW>
__global__ void __launch_bounds__(256) gated_pairs_kernel(GatedArgs g) {
    pdl_trigger();
    pdl_wait();
    const int blk = blockIdx.z, m0 = blockIdx.x * GT_M, n0 = blockIdx.y * GT_N, n = g.n;
    const float *A = g.u + (size_t)blk * n;
    const TW *wr = (const TW *)g.w_r + (size_t)blk * n * n, *wi = (const TW *)g.w_i + (size_t)blk * n * n;
    float zr[16], zi[16];
    if constexpr (OnTensorCores<TW>::value) tile_product_split<true>(A, (size_t)g.C, g.T, wr, wi, (size_t)n, n, n, m0, n0, zr, zi);
    else tile_product<true>(A, (size_t)g.C, nullptr, g.T, wr, wi, (size_t)n, n, n, m0, n0, zr, zi);
#pragma unroll
    for (int e = 0; e < 16; ++e) {
        int r, k;
        tile_at<TW>(e, &r, &k);
        const int t = m0 + r;
        if (t >= g.T || n0 + k >= n) continue;
        const int c = blk * n + n0 + k;
        const size_t at = (size_t)t * g.C + c;
        gated_pair(zr[e] + g.b_r[c], zi[e] + g.b_i[c], g.rate[c], g.u[at], g.a + at, g.b + at);
    }
}

constexpr int GS_THREADS = 128, GS_AHEAD = 8;

// rows [first, last) of channel c from state s; OUT: their outputs; else the product of their decays into *prod
template <typename T, bool OUT>
__device__ __forceinline__ float gated_walk(const GatedArgs &g, int c, int first, int last, float s, float *prod) {
    const float yb = OUT && g.y_bias != nullptr ? g.y_bias[c] : 0.f;
    float p = 1.f;
    float a[2][GS_AHEAD], b[2][GS_AHEAD], y[2][GS_AHEAD];       // two groups of rows that take turns: one on its way, one being walked
    auto fetch = [&](int t0, float (&fa)[GS_AHEAD], float (&fb)[GS_AHEAD], float (&fy)[GS_AHEAD]) {
#pragma unroll
        for (int j = 0; j < GS_AHEAD; ++j) {
            const size_t t = min(t0 + j, last - 1);
            fa[j] = g.a[t * g.C + c];
            fb[j] = g.b[t * g.C + c];
            fy[j] = OUT ? g.y[t * g.ld_y + c] : 0.f;
        }
    };
    auto walk = [&](int t0, const float (&fa)[GS_AHEAD], const float (&fb)[GS_AHEAD], const float (&fy)[GS_AHEAD]) {
#pragma unroll
        for (int j = 0; j < GS_AHEAD; ++j) {
            if (t0 + j >= last) break;
            s = fmaf(fa[j], s, fb[j]);
            if (OUT) ((T *)g.out)[(size_t)(t0 + j) * g.C + c] = from_f32<T>(s * block_act(g.act, fy[j] + yb));
            else p *= fa[j];
        }
    };
    fetch(first, a[0], b[0], y[0]);
    for (int t0 = first; t0 < last; t0 += 2 * GS_AHEAD) {
        if (t0 + GS_AHEAD < last) fetch(t0 + GS_AHEAD, a[1], b[1], y[1]);
        walk(t0, a[0], b[0], y[0]);
        if (t0 + 2 * GS_AHEAD < last) fetch(t0 + 2 * GS_AHEAD, a[0], b[0], y[0]);
        if (t0 + GS_AHEAD < last) walk(t0 + GS_AHEAD, a[1], b[1], y[1]);
    }
    if (!OUT) *prod = p;
    return s;
}

// whose piece p is: (the request's first piece, its pieces, the request)
__device__ __forceinline__ int3 gated_piece_of(const GatedArgs &g, int p) {
    for (int i = 0; i < g.n_piece_reqs; ++i) {
        const int first = g.piece_reqs[3 * i + 1], n = g.piece_reqs[3 * i + 2];
        if (p >= first && p < first + n) return make_int3(first, n, g.piece_reqs[3 * i]);
    }
    return make_int3(p, 1, 0);
}

template <typename T>
__global__ void __launch_bounds__(GS_THREADS) gated_scan_kernel(GatedArgs g) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * GS_THREADS + threadIdx.x, item = blockIdx.y;
    if (c >= g.C) return;
    if (item < g.n_direct) {
        const int req = g.direct ? g.direct[item] : item;
        float *S = g.state + (size_t)g.slot_ids[req] * g.C + c;
        *S = gated_walk<T, true>(g, c, g.req_start[req], g.req_start[req + 1], *S, nullptr);
        return;
    }
    const int p = item - g.n_direct, first = g.pieces[2 * p], last = first + g.pieces[2 * p + 1];
    const int3 of = gated_piece_of(g, p);
    if (p == of.x) {
        float *S = g.state + (size_t)g.slot_ids[of.z] * g.C + c;
        const float s = gated_walk<T, true>(g, c, first, last, *S, nullptr);
        g.piece_end[(size_t)p * g.C + c] = s;
        if (of.y == 1) *S = s;
    } else {
        float prod;
        g.piece_end[(size_t)p * g.C + c] = gated_walk<T, false>(g, c, first, last, 0.f, &prod);
        g.piece_prod[(size_t)p * g.C + c] = prod;
    }
}

template <typename T>
__global__ void __launch_bounds__(GS_THREADS) gated_finish_kernel(GatedArgs g) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * GS_THREADS + threadIdx.x, p = blockIdx.y;
    if (c >= g.C) return;
    const int3 of = gated_piece_of(g, p);
    if (p == of.x) return;
    float s = g.piece_end[(size_t)of.x * g.C + c];
    for (int q0 = of.x + 1; q0 < p; q0 += GS_AHEAD) {
        float e[GS_AHEAD], d[GS_AHEAD];
#pragma unroll
        for (int j = 0; j < GS_AHEAD; ++j) {
            const size_t q = min(q0 + j, p - 1);
            e[j] = g.piece_end[q * g.C + c];
            d[j] = g.piece_prod[q * g.C + c];
        }
#pragma unroll
        for (int j = 0; j < GS_AHEAD; ++j)
            if (q0 + j < p) s = fmaf(d[j], s, e[j]);
    }
    const int first = g.pieces[2 * p], last = first + g.pieces[2 * p + 1];
    s = gated_walk<T, true>(g, c, first, last, s, nullptr);
    if (p == of.x + of.y - 1) g.state[(size_t)g.slot_ids[of.z] * g.C + c] = s;
}

// One row a request (row t is request t's): GR_ROWS rows and GR_CHANNELS channels of one part a block.  The rows' inputs wait in
// shared memory; a warp takes a channel at a time, its lanes the row of both matrices; then lane r does row r's step.
constexpr int GR_ROWS = 8, GR_CHANNELS = 16;

template <typename T, int ROWS>
__device__ __forceinline__ void gated_rows_body(const GatedArgs &g, const float *rows_u, int t0, int live, int blk, int c_first) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n = g.n;
    constexpr int V = Vec16<T>::N;
    const bool vec = n % V == 0 && n % 4 == 0 && ((uintptr_t)g.w_r | (uintptr_t)g.w_i) % 16 == 0;
    for (int k = c_first + warp; k < min(n, c_first + GR_CHANNELS); k += 8) {
        const T *wr = (const T *)g.w_r + ((size_t)blk * n + k) * n, *wi = (const T *)g.w_i + ((size_t)blk * n + k) * n;
        float zr[ROWS], zi[ROWS];
#pragma unroll
        for (int r = 0; r < ROWS; ++r) { zr[r] = 0.f; zi[r] = 0.f; }
        if (vec) {
#pragma unroll 2
            for (int j = lane * V; j < n; j += 32 * V) {
                float fr[V], fi[V];
                unpack16<T>(*reinterpret_cast<const uint4 *>(wr + j), fr);
                unpack16<T>(*reinterpret_cast<const uint4 *>(wi + j), fi);
#pragma unroll
                for (int r = 0; r < ROWS; ++r)
#pragma unroll
                    for (int v = 0; v < V; v += 4) {
                        const float4 x = *reinterpret_cast<const float4 *>(rows_u + (size_t)r * n + j + v);
                        zr[r] = fmaf(fr[v + 3], x.w, fmaf(fr[v + 2], x.z, fmaf(fr[v + 1], x.y, fmaf(fr[v], x.x, zr[r]))));
                        zi[r] = fmaf(fi[v + 3], x.w, fmaf(fi[v + 2], x.z, fmaf(fi[v + 1], x.y, fmaf(fi[v], x.x, zi[r]))));
                    }
            }
        } else {
            for (int j = lane; j < n; j += 32)
#pragma unroll
                for (int r = 0; r < ROWS; ++r) {
                    zr[r] = fmaf(to_f32(wr[j]), rows_u[(size_t)r * n + j], zr[r]);
                    zi[r] = fmaf(to_f32(wi[j]), rows_u[(size_t)r * n + j], zi[r]);
                }
        }
        float mr = 0.f, mi = 0.f;       // lane r: row r's sums
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            const float a = warp_sum(zr[r]), b = warp_sum(zi[r]);
            if (lane == r) { mr = a; mi = b; }
        }
        if (lane < live) {
            const int t = t0 + lane, c = blk * n + k;
            float a, b;
            gated_pair(mr + g.b_r[c], mi + g.b_i[c], g.rate[c], rows_u[(size_t)lane * n + k], &a, &b);
            float *S = g.state + (size_t)g.slot_ids[t] * g.C + c;
            const float s = fmaf(a, *S, b);
            *S = s;
            ((T *)g.out)[(size_t)t * g.C + c] = from_f32<T>(s * block_act(g.act, g.y[(size_t)t * g.ld_y + c] + (g.y_bias ? g.y_bias[c] : 0.f)));
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) gated_rows_kernel(GatedArgs g) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float rows_u[];     // [rows][n], rows 1, 2, 4 or 8
    const int blk = blockIdx.y, t0 = blockIdx.z * GR_ROWS, live = min(GR_ROWS, g.T - t0), n = g.n;
    const int rows = live <= 1 ? 1 : (live <= 2 ? 2 : (live <= 4 ? 4 : 8));
    for (int i = threadIdx.x; i < rows * n; i += 256) {
        const int r = i / n;
        rows_u[i] = r < live ? g.u[(size_t)(t0 + r) * g.C + (size_t)blk * n + i - r * n] : 0.f;
    }
    __syncthreads();
    const int c_first = blockIdx.x * GR_CHANNELS;
    if (rows == 1) gated_rows_body<T, 1>(g, rows_u, t0, live, blk, c_first);
    else if (rows == 2) gated_rows_body<T, 2>(g, rows_u, t0, live, blk, c_first);
    else if (rows == 4) gated_rows_body<T, 4>(g, rows_u, t0, live, blk, c_first);
    else gated_rows_body<T, 8>(g, rows_u, t0, live, blk, c_first);
}

// floats of scratch that a step of T rows with n_pieces pieces needs
JK_EXPORT long long jk_gated_recurrence_scratch_floats(int T, int C, int n_pieces) { return 2LL * T * C + 2LL * n_pieces * C; }
// kernels that a call launches
JK_EXPORT int jk_gated_recurrence_launches(int T, int nreq, int n, int n_pieces) {
    return T == nreq && T <= 64 && (size_t)n * GR_ROWS * 4 <= 200 * 1024 ? 1 : (n_pieces > 0 ? 3 : 2);
}

JK_EXPORT int jk_gated_recurrence(const float *u, const void *w_r, const void *w_i, const float *b_r, const float *b_i, const float *rate, const float *y,
                                  int ld_y, const float *y_bias, int act, float *state, const int *req_start, const int *slot_ids, int nreq, void *out,
                                  int dtype, int T, int C, int blocks, const int *direct, int n_direct, const int *pieces, int n_pieces,
                                  const int *piece_reqs, int n_piece_reqs, float *scratch, long long scratch_floats, cudaStream_t stream) {
    if (T == 0 || nreq == 0) return JK_OK;
    JK_REQUIRE(u && w_r && w_i && b_r && b_i && rate && y && state && req_start && slot_ids && out, "gated_recurrence: an argument is missing");
    JK_REQUIRE(C > 0 && blocks > 0 && C % blocks == 0 && blocks <= 65535, "gated_recurrence: %d channels in %d parts", C, blocks);
    GatedArgs g{u, w_r, w_i, b_r, b_i, rate, y, ld_y, y_bias, act, state, req_start, slot_ids, out, T, C, blocks, C / blocks,
                nullptr, nullptr, nullptr, nullptr, direct, pieces, piece_reqs, n_direct, n_pieces, n_piece_reqs};
    if (jk_gated_recurrence_launches(T, nreq, g.n, n_pieces) == 1) {
        const size_t smem = sizeof(float) * (size_t)(T <= 1 ? 1 : (T <= 2 ? 2 : (T <= 4 ? 4 : 8))) * g.n;
        const dim3 grid((g.n + GR_CHANNELS - 1) / GR_CHANNELS, blocks, (T + GR_ROWS - 1) / GR_ROWS);
#define LAUNCH(TT)                                                                                                                     \
    do {                                                                                                                               \
        if (smem > 46 * 1024) cudaFuncSetAttribute(gated_rows_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
        jk_launch(gated_rows_kernel<TT>, grid, dim3(256), smem, stream, g);                                                            \
    } while (0)
        BLOCKS_BY_DTYPE(dtype, "gated_rows", LAUNCH);
#undef LAUNCH
        JK_CHECK_LAUNCH("gated_rows");
        return JK_OK;
    }
    if (n_pieces == 0 && direct == nullptr && n_direct <= 0) g.n_direct = nreq;       // no lists: every request is one item
    JK_REQUIRE(g.n_direct >= 0 && n_pieces >= 0 && g.n_direct + n_pieces > 0 && g.n_direct + n_pieces <= 65535, "gated_recurrence: %d and %d work items", n_direct, n_pieces);
    JK_REQUIRE(n_pieces == 0 || (pieces && piece_reqs && n_piece_reqs > 0), "gated_recurrence: pieces without their lists");
    JK_REQUIRE(scratch && scratch_floats >= jk_gated_recurrence_scratch_floats(T, C, n_pieces), "gated_recurrence: %lld floats of scratch are too few", scratch_floats);
    g.a = scratch; g.b = g.a + (size_t)T * C; g.piece_end = g.b + (size_t)T * C; g.piece_prod = g.piece_end + (size_t)n_pieces * C;
    const dim3 tiles((T + GT_M - 1) / GT_M, (g.n + GT_N - 1) / GT_N, blocks);
    const int groups = (C + GS_THREADS - 1) / GS_THREADS;
#define LAUNCH(TT)                                                                                                                   \
    jk_launch(gated_pairs_kernel<TT>, tiles, dim3(256), 0, stream, g);                                                               \
    jk_launch(gated_scan_kernel<TT>, dim3(groups, g.n_direct + n_pieces), dim3(GS_THREADS), 0, stream, g);                           \
    if (n_pieces > 0) jk_launch(gated_finish_kernel<TT>, dim3(groups, n_pieces), dim3(GS_THREADS), 0, stream, g)
    BLOCKS_BY_DTYPE(dtype, "gated_recurrence", LAUNCH);
#undef LAUNCH
    JK_CHECK_LAUNCH("gated_recurrence");
    return JK_OK;
}
