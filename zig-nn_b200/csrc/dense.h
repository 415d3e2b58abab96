// Mechanisms of decoders whose weights are plain bf16 matrices (internal declarations): linears, norms with the
// residual sum, grouped-query and latent attention over a cache, recurrences with a matrix state, and the mixture of
// experts. Every launcher takes `f32`: false = activations (and the key / value cache) are bf16,
// true = everything is f32. Accumulators, norms, scores, routers, the residual and recurrent state are f32 in both.
#pragma once

#include <cuda_bf16.h>

#include "zq_internal.h"

namespace zq {

using bf16 = __nv_bfloat16;

inline uint32_t pad_to(uint32_t n, uint32_t m) { return (n + m - 1) / m * m; }
// Row pitch of weights and of activation rows that feed a linear: zeros beyond the real columns.
inline uint32_t pad64(uint32_t n) { return pad_to(n, 64); }
inline size_t act_bytes(bool f32) { return f32 ? 4 : 2; }
constexpr float kLog2e = 1.4426950408889634f;

// [rows][kp] bf16 on the device, kp = pad64(k), zero beyond column k.
struct DenseWeight {
    bf16* w = nullptr;
    uint32_t rows = 0, k = 0, kp = 0;
};

// A gate and an up matrix of ff rows each are stacked as ONE matrix of 2 * pad64(ff) rows in blocks of 32: 16 gate
// rows, then the 16 up rows of the same features (both sit in one warp of a tensor-core epilogue).
__host__ __device__ inline uint32_t glu_row(uint32_t feature, bool up) {
    return (feature >> 4) * 32u + (feature & 15u) + (up ? 16u : 0u);
}
enum GluKind { GLU_SILU = 0, GLU_CLAMPED = 1 };
struct GluSpec {
    int kind = GLU_SILU;
    float limit = 0.0f;  // GLU_CLAMPED
};

// One of the products of a launch: rows [w_row, w_row + rows) of the weight times the T activation rows from x_row
// on, written to columns y_col... of the T output rows.
struct LinGroup {
    uint32_t w_row, rows, x_row, y_col;
};
constexpr uint32_t kMaxLinGroups = 8;
struct LinGroups {
    LinGroup g[kMaxLinGroups];
    uint32_t n;
};
inline LinGroups one_group(uint32_t rows) {
    LinGroups G{};
    G.n = 1;
    G.g[0] = LinGroup{0, rows, 0, 0};
    return G;
}

// A product may come as several addends (the K dimension cut over CTAs): y = sum of `n` arrays `stride` floats apart.
struct Addends {
    uint32_t n = 1;
    size_t stride = 0;
};
// y[t][y_col + j] = sum_k x[x_row + t][k] * W[w_row + j][k], f32 out. x: activation rows of pitch W.kp, x_rows of them.
// add != null: y has room for y_floats floats and the result may be left as addends (one group only).
int launch_dense_linear(const DenseWeight& W, const LinGroups& G, const void* x, uint32_t x_rows, uint32_t T, float* y,
                        uint32_t y_stride, bool f32, cudaStream_t st, Addends* add = nullptr, size_t y_floats = 0);
// out[t][f] = glu(gate row f . x[t], up row f . x[t]) for the pad64(ff) features of an interleaved weight.
int launch_dense_glu(const DenseWeight& W, const void* x, uint32_t T, void* out, GluSpec glu, bool f32, cudaStream_t st);

// Chosen experts of T tokens, `top` pairs (token, expert) per token, and an optional shared expert for every token.
struct MoeWeights {
    DenseWeight gate_up;         // [experts * 2 * ffp][kp], interleaved per expert
    DenseWeight down;            // [experts * width][ffp]
    DenseWeight shared_gate_up;  // empty without a shared expert
    DenseWeight shared_down;
    uint32_t experts = 0, top = 0, ffp = 0, shared_ffp = 0, width = 0;
    GluSpec glu, shared_glu;
    bool scale_input = true;     // a pair's weight multiplies the expert's input; otherwise its output (add_norm)
};
// What a routed batch looks like in device memory.
struct MoeRouting {
    int32_t* ids;       // [T * top] expert of pair t * top + k
    float* weights;     // [T * top] its weight
    int32_t* place;     // [T * top] row of the pair in expert order (many tokens)
    int32_t* source;    // [T * top] inverse: pair at that row
    int32_t* offsets;   // [experts + 1] first row of each expert
    int32_t* tiles;     // [2 * kMoeMaxTiles + 1]: count, then (expert, first row) per tile of `bn` rows
};
constexpr uint32_t kMoeMaxTiles = 4096;

// Few tokens: one GEMV per pair (and per token for the shared expert). parts: [T * top + T] rows of `width`. The rows are
// not scaled by an output weight.
int launch_moe_pairs(const MoeWeights& M, const MoeRouting& R, const void* x, uint32_t T, void* hidden, float* parts,
                     bool f32, cudaStream_t st);
// Many tokens, bf16: xs = the pairs' inputs in expert order (already scaled), grouped tensor-core products.
int launch_moe_grouped(const MoeWeights& M, const MoeRouting& R, const bf16* xs, uint32_t T, uint32_t bn, bf16* hidden,
                       float* parts, cudaStream_t st);
// bf16 tensor-core product (gemm_bf16.cu); GLU epilogue when `glu` is given, else f32 out.
int launch_gemm_bf16(const DenseWeight& W, const LinGroups& G, const bf16* x, uint32_t x_rows, uint32_t T, float* y,
                     uint32_t y_stride, bf16* glu_out, uint32_t glu_stride, const GluSpec* glu, cudaStream_t st,
                     Addends* add = nullptr, size_t y_floats = 0);
// The product of [heads * d0 | heads * d1] weight rows, bf16, head by head to two arrays [T][heads][pitch]: x rows of
// x_pitch values (multiple of 8) that may hold finite values beyond W.k.
struct HeadSplit {
    bf16 *out0, *out1;
    uint32_t heads, d0, d1, pitch0, pitch1;
};
int launch_gemm_bf16_heads(const DenseWeight& W, const bf16* x, uint32_t x_pitch, uint32_t x_rows, uint32_t T,
                           const HeadSplit& split, cudaStream_t st);
constexpr uint32_t kDenseGemmMinRows = 9;  // fewer activation rows take the GEMV

// ---- norms, embedding, token shift (dense_ops.cu) --------------------------------------------------------------
struct AddNormArgs {
    // 1. what is added to the residual stream x [rows][width] (all optional)
    const bf16* embed;       // x = embed[tokens[r]] * embed_scale (pitch embed_kp), normed with embed_w if that is given
    const int32_t* tokens;
    uint32_t embed_kp;
    float embed_scale;
    const float* embed_w;
    const float* y;          // the sum of: y, possibly as addends,
    Addends y_add;
    const float* y2;         // y2 likewise (two sublayers that read the same h),
    Addends y2_add;
    const float* parts;      // and the token's `top` rows of parts (+ its shared row)
    const float* part_w;     // weight of pair p (null: 1)
    const int32_t* place;    // row of pair p (null: p)
    uint32_t top;
    const float* shared;     // [rows][width]
    const float* shared_gate;  // times sigmoid(element r * gate_stride); null: times 1
    uint32_t gate_stride;
    const float* post_w;     // x += norm(sum) * post_w; null: x += sum
    float* x;
    // 2. what is computed from it (optional): h = norm(x) * pre_w
    const float* pre_w;
    void* h;                 // activation rows, pitch hp
    float* h32;              // the same in f32, pitch width
    const int32_t* rows_from;  // row r of the outputs comes from row rows_from[r] of x (no addition then)
    // 3. token shift of a decode step: mix_s = h + (h_prev - h) * mu_s; h_prev of the row's slot, replaced by h
    const float* mu;         // [n_mix][width]
    float* prev;             // [slots][width]
    const int32_t* slots;
    void* mix;               // [n_mix][mix_rows] activation rows
    uint32_t n_mix, mix_rows;
    uint32_t width, hp;
    float eps;
};
int launch_add_norm(const AddNormArgs& a, uint32_t rows, bool f32, cudaStream_t st);
// Token shift of `rows` consecutive tokens of one sequence: h32 [rows][width], the token ahead of row 0 is prev[slots[0]].
int launch_token_shift(const float* h32, const float* mu, const float* prev, const int32_t* slots, uint32_t n_mix,
                       uint32_t rows, uint32_t mix_rows, uint32_t width, void* mix, bool f32, cudaStream_t st);

// ---- attention (dense_attention.cu) ----------------------------------------------------------------------------
struct GqaShape {
    uint32_t heads, kv_heads, dim, vdim, dimp, vdimp, ctx, slots;  // dimp / vdimp: cache pitch per head, multiples of 16
};
struct QkvPostArgs {
    GqaShape s;
    const float* qkv;        // [rows][heads * dim | kv_heads * dim | kv_heads * vdim]
    const float *q_norm, *k_norm;  // plain RMS-norm weights [dim]
    float eps, temp_coef, temp_every;  // query temperature; temp_every = 0: none
    const float* vmix;       // v = (1 - *vmix) v + *vmix * v_first (null: as projected)
    float* v_first;          // [rows][kv_heads * vdim]; written when vmix is null and v_first is not
    void *q, *kc, *vc;       // q [rows][heads][dimp]; caches [slots][ctx][kv_heads][dimp / vdimp]
    const int32_t *pos, *slots;
};
int launch_qkv_post(const QkvPostArgs& a, uint32_t rows, bool f32, cudaStream_t st);
// launch_qkv_post and launch_gqa_attention of the same rows; a decode step in bf16 does both in one kernel.
int launch_gqa_layer(const QkvPostArgs& a, void* out, uint32_t out_pitch, float scale, uint32_t rows, bool one_sequence,
                     uint32_t pos0, void* work, bool f32, cudaStream_t st);
// Causal softmax attention of every row (position pos[r], slot slots[r]) over its slot's cache, the rows' own keys
// included. out: activation rows of pitch out_pitch = pad64(heads * vdim). one_sequence: the rows are consecutive
// tokens of slots[0] and pos0 is pos[0] (known on the host). work: gqa_work_bytes.
size_t gqa_work_bytes(const GqaShape& s, uint32_t max_rows);
int launch_gqa_attention(const GqaShape& s, const void* q, const void* kc, const void* vc, void* out, uint32_t out_pitch,
                         float scale, const int32_t* pos, const int32_t* slots, uint32_t rows, bool one_sequence,
                         uint32_t pos0, void* work, bool f32, cudaStream_t st);

// The form without tiles, any number of rows: dimp is the pitch of a query and a key, vdimp that of a value (which may be a
// view of the key rows).
int launch_gqa_plain(const GqaShape& s, const void* q, const void* kc, const void* vc, void* out, uint32_t out_pitch, float scale,
                     const int32_t* pos, const int32_t* slots, uint32_t rows, bool f32, cudaStream_t st);

// The prefill form on tcgen05 (dense_attention_tc.cu); ZQ_ERR_UNSUPPORTED where its tensor maps do not exist.
int launch_gqa_prefill_tc(const GqaShape& s, const bf16* q, const bf16* kc, const bf16* vc, bf16* out, uint32_t out_pitch,
                          float scale2, const int32_t* slots, uint32_t rows, uint32_t pos0, cudaStream_t st);

// ---- decayed outer-product recurrence (dense_wkv.cu) --------------------------------------------------------------
struct WkvArgs {
    uint32_t heads, dim, rank, rank_p, ld;  // ld: pitch of rkvg
    const float* rkvg;       // [rows][r | k | v | g | w1 output (rank)], heads * dim each, pitch ld
    const bf16* w2;          // [heads * dim][rank_p]
    const float *w0, *u, *norm;
    float eps;
    float* state;            // [slots][heads][dim][dim]
    const int32_t* slots;
    void* out;               // activation rows of pitch out_pitch = pad64(heads * dim)
    uint32_t out_pitch;
    const float* h32;        // many tokens: the last row becomes prev[slots[0]]
    float* prev;
    uint32_t width;
    float* decay;            // scratch, many tokens: [rows][heads * dim]
    float* chunk;            // scratch, many tokens: wkv_chunk_floats
};
size_t wkv_chunk_floats(uint32_t heads, uint32_t dim, uint32_t max_rows);
int launch_wkv(const WkvArgs& a, uint32_t rows, bool one_sequence, bool f32, cudaStream_t st);

// ---- recurrences with a matrix state behind per-token gates (dense_state.cu) ----------------------------------------
// Per head a state S [dim][vdim] in f32; then every head's o over its root mean square, times norm, times sigmoid(gate).
//   memory   S <- a S + b k v^T, n <- a n + b k under a running maximum m of the log gates, o = S^T q / size(n . q)
//   delta    S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q
struct MemoryArgs {
    uint32_t heads, dim, vdim, ld;
    const float* in;         // [rows][q | k | v | gate | i | f], pitch ld
    const float *i_bias, *f_bias;  // [heads]
    float gate_cap;
    const float* norm;       // [heads * vdim]
    float eps;
    float *S, *n, *m;        // [slots][heads][dim][vdim], [slots][heads][dim], [slots][heads]
    const int32_t* slots;
    void* out;               // activation rows of pitch out_pitch = pad64(heads * vdim)
    uint32_t out_pitch;
    float* work;             // many tokens: memory_work_floats
};
size_t memory_work_floats(uint32_t heads, uint32_t dim, uint32_t vdim, uint32_t max_rows);
int launch_memory(const MemoryArgs& a, uint32_t rows, bool one_sequence, bool f32, cudaStream_t st);

struct DeltaArgs {
    uint32_t heads, kv_heads, dim, vdim, taps, a_rank, g_rank, ld;
    const float* in;         // [rows][q | k | v | beta | a1 output | g1 output], pitch ld
    const float* conv;       // [channels of q | k | v][taps], the last tap is the current token's
    const float *A_log, *dt_bias;  // [heads], [heads * dim]
    DenseWeight low;         // [heads * dim rows over the a1 output | heads * vdim rows over the g1 output]
    const float* norm;       // [vdim]
    float eps;
    float* S;                // [slots][heads][dim][vdim]
    float* ring;             // [slots][taps][channels]: inputs of the convolution, token p at place p % taps (unused with 1 tap)
    const int32_t *pos, *slots;
    void* out;
    uint32_t out_pitch;
    float* work;             // many tokens: delta_work_floats
    uint32_t max_rows;       // rows that work is made for
};
size_t delta_work_floats(const DeltaArgs& a, uint32_t max_rows);
int launch_delta(const DeltaArgs& a, uint32_t rows, bool one_sequence, bool f32, cudaStream_t st);

// ---- attention over a cache of latents (dense_latent.cu) ------------------------------------------------------------
// A cache row holds the normed latent [rank] and the rotated key part [rot] that all heads share, keyp = pad16 of both.
// Key of a head: [W_uk latent | key part], value: W_uv latent. Decoding and short portions fold W_uk into the query and
// W_uv behind the weighted sum, so that a row of the cache is read once for all heads; longer portions (bf16) write the
// heads' keys and values out and take the grouped-query kernels.
struct LatentShape {
    uint32_t heads, dim, rot, vdim, rank, keyp, ctx, slots;
};
struct LatentArgs {
    LatentShape s;
    const float* in;         // [rows][heads * (dim + rot) | rank + rot if own], pitch ld
    uint32_t ld;
    bool own;                // the layer writes the cache (otherwise another one has)
    const float* norm;       // [rank], with own
    float eps, scale;
    const float* freq;       // [rot / 2] angle per position
    DenseWeight up;          // [heads * dim | heads * vdim] rows over rank
    void* cache;             // [slots][ctx][keyp] activations
    const int32_t *pos, *slots;
    uint32_t slot0;          // one_sequence: slots[0] (known on the host)
    void* out;               // activation rows of pitch out_pitch = pad64(heads * vdim)
    uint32_t out_pitch;
    void* work;              // latent_work_bytes
    uint32_t max_rows;
};
size_t latent_work_bytes(const LatentShape& s, uint32_t max_rows, bool f32);
int launch_latent(const LatentArgs& a, uint32_t rows, bool one_sequence, uint32_t pos0, bool f32, cudaStream_t st);

// ---- mixture of experts (dense_ops.cu) ----------------------------------------------------------------------------
// z [rows][z_stride] router logits (+ bias) -> ids of the `top` largest and their weights
enum RouteKind { ROUTE_SIGMOID = 0, ROUTE_SOFTMAX = 1 };  // own sigmoid; softmax over the chosen ones
int launch_route(const float* z, uint32_t z_stride, uint32_t experts, uint32_t top, const float* bias, int kind,
                 const MoeRouting& R, uint32_t rows, cudaStream_t st);
// Expert order of the pairs, tiles of bn rows, and xs[place] = h[token] (times the pair's weight).
int launch_moe_plan(const MoeRouting& R, uint32_t experts, uint32_t top, uint32_t rows, uint32_t bn, const bf16* h,
                    uint32_t hp, bool scale_input, bf16* xs, cudaStream_t st);

#ifdef __CUDACC__
template <typename TA>
__device__ __forceinline__ TA to_act(float v);
template <>
__device__ __forceinline__ float to_act<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 to_act<bf16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float from_act(float v) { return v; }
__device__ __forceinline__ float from_act(bf16 v) { return __bfloat162float(v); }

__device__ __forceinline__ float bf16_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t u) { return __uint_as_float(u & 0xFFFF0000u); }
__device__ __forceinline__ void unpack8(const uint4& u, float (&f)[8]) {
    f[0] = bf16_lo(u.x); f[1] = bf16_hi(u.x); f[2] = bf16_lo(u.y); f[3] = bf16_hi(u.y);
    f[4] = bf16_lo(u.z); f[5] = bf16_hi(u.z); f[6] = bf16_lo(u.w); f[7] = bf16_hi(u.w);
}
// eight consecutive activations from a 16-byte aligned address
__device__ __forceinline__ void load8(const bf16* p, float (&f)[8]) { unpack8(*reinterpret_cast<const uint4*>(p), f); }
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float glu_value(float g, float u, int kind, float limit) {
    if (kind == GLU_CLAMPED) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g * sigmoid_f(1.702f * g) * (u + 1.0f);
    }
    return g * sigmoid_f(g) * u;
}
__device__ __forceinline__ float warp_sum_f(float v) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, off);
    return v;
}
// ---- steps between the projections and the attention of one row, a warp per head ----
// Factor of the RMS norm of a head's `dim` values.
__device__ __forceinline__ float head_norm_factor(const float* v, uint32_t dim, float eps, uint32_t lane) {
    float ss = 0.0f;
    for (uint32_t i = lane; i < dim; i += 32) ss = fmaf(v[i], v[i], ss);
    return 1.0f / sqrtf(warp_sum_f(ss) / (float)dim + eps);
}
__device__ __forceinline__ float query_temperature(uint32_t pos, float coef, float every) {
    return every > 0.0f ? 1.0f + coef * logf(floorf((float)(pos + 1) / every) + 1.0f) : 1.0f;
}
// out[i] = v[i] * norm factor * w[i] * temp for i < dim, zeros up to dimp
template <typename TA>
__device__ __forceinline__ void norm_head(const float* v, const float* w, uint32_t dim, uint32_t dimp, float eps, float temp,
                                          TA* out, uint32_t lane) {
    const float f = head_norm_factor(v, dim, eps, lane);
    for (uint32_t i = lane; i < dimp; i += 32) out[i] = to_act<TA>(i < dim ? v[i] * f * w[i] * temp : 0.0f);
}
// The values of a head, mixed with those of the first mixing layer or kept for later layers.
__device__ __forceinline__ float mixed_value(float v, const float* vmix, float* first, uint32_t i) {
    if (vmix) return (1.0f - *vmix) * v + *vmix * first[i];
    if (first) first[i] = v;
    return v;
}
// Sum over the block in a fixed order; every thread gets it. red: 33 floats, reusable after the call.
__device__ __forceinline__ float block_sum_f(float v, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    v = warp_sum_f(v);
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float t = lane < nw ? red[lane] : 0.0f;
    t = warp_sum_f(t);
    __syncthreads();
    return t;
}
#endif

}  // namespace zq
