// The recurrence S_t = diag(w_t) S_(t-1) + k_t v_t^T with read-out o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t, per
// head, state in f32; then every head's o over its root mean square, times a weight and a gate.
//
// A thread holds RPT key rows of one value column of the state; four threads of a warp hold one column, a CTA one
// head. A decode step is one such CTA per (sequence, head), the decays computed in its prologue. Many tokens of
// one sequence are cut into chunks: (1) every chunk's own contribution and decay product from a zero state, all
// chunks at once; (2) the chunks' starting states by a short scan over them; (3) every chunk again with its starting
// state, now with the read-out. Chunk borders are counted from the portion's first token; the state stays f32.
#include "dense.h"

namespace zq {
namespace {

constexpr uint32_t kWkvTile = 16;    // tokens staged in shared memory at a time
constexpr uint32_t kWkvChunk = 64;   // tokens per chunk
constexpr uint32_t kWkvMaxDim = 256;

struct WkvParams {
    WkvArgs a;
    uint32_t rows, chunk_len, n_chunks;
    bool per_row;          // every row is its own sequence (decode)
};

// decay[t][c] = exp(-exp(w0[c] + sum_q w2[c][q] tanh(x[t][q]))), x = the w1 columns of rkvg: a CTA takes 64 channels of
// 16 tokens.
__global__ void __launch_bounds__(256)
wkv_decay_kernel(const __grid_constant__ WkvParams p) {
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    pdl_wait();
    const WkvArgs& a = p.a;
    const uint32_t HD = a.heads * a.dim, R = a.rank, c0 = blockIdx.x * 64, t0 = blockIdx.y * 16;
    float* xs = sm;                 // [16][R]
    float* ws = sm + 16 * R;        // [64][R + 1]
    for (uint32_t i = threadIdx.x; i < 16 * R; i += 256) {
        const uint32_t t = t0 + i / R;
        xs[i] = t < p.rows ? tanhf(a.rkvg[(size_t)t * a.ld + 4 * HD + i % R]) : 0.0f;
    }
    for (uint32_t i = threadIdx.x; i < 64 * R; i += 256) {
        const uint32_t c = c0 + i / R;
        ws[(i / R) * (R + 1) + i % R] = c < HD ? __bfloat162float(a.w2[(size_t)c * a.rank_p + i % R]) : 0.0f;
    }
    __syncthreads();
    const uint32_t c = threadIdx.x & 63, tq = threadIdx.x >> 6;
    if (c0 + c >= HD) return;
    float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    for (uint32_t q = 0; q < R; ++q) {
        const float w = ws[c * (R + 1) + q];
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i] = fmaf(w, xs[(tq * 4 + i) * R + q], acc[i]);
    }
    const float w0 = a.w0[c0 + c];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const uint32_t t = t0 + tq * 4 + i;
        if (t < p.rows) a.decay[(size_t)t * HD + c0 + c] = expf(-expf(acc[i] + w0));
    }
}

// OUT: read-out and epilogue; otherwise the chunk's contribution from a zero state and its decay product.
template <int RPT, bool OUT, typename TA>
__global__ void __launch_bounds__(RPT * 16)
wkv_kernel(const __grid_constant__ WkvParams p) {
    constexpr uint32_t PS = RPT + 4;       // pitch of a thread's rows in the staged vectors: no bank conflicts
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    const WkvArgs& a = p.a;
    const uint32_t D = a.dim, HD = a.heads * D, h = blockIdx.x, chunk = blockIdx.y;
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const uint32_t part = lane & 3, col = warp * 8 + (lane >> 2);
    float* rs = sm;                              // [tile][4 * PS]
    float* ks = rs + kWkvTile * 4 * PS;
    float* ws = ks + kWkvTile * 4 * PS;
    float* vs = ws + kWkvTile * 4 * PS;          // [tile][D]
    float* os = vs + kWkvTile * D;               // [tile][D]
    float* bs = os + kWkvTile * D;               // [tile]
    float* us = bs + kWkvTile;                   // [4 * PS]
    float* lo = us + 4 * PS;                     // [rank] (decode)
    auto place = [&](uint32_t i) { return (i / RPT) * PS + i % RPT; };
    pdl_wait();

    const uint32_t t_begin = chunk * p.chunk_len, t_end = min(p.rows, t_begin + p.chunk_len);
    const uint32_t slot = (uint32_t)a.slots[p.per_row ? chunk : 0];
    const size_t state_at = ((size_t)slot * a.heads + h) * D * D;
    const size_t chunk_state = (size_t)p.n_chunks * a.heads;  // [chunk][head] states, then [chunk][head][D] decays
    float* cstate = a.chunk + ((size_t)chunk * a.heads + h) * D * D;
    const bool from_chunk = OUT && !p.per_row && p.n_chunks > 1;

    float S[RPT], dp[OUT ? 1 : RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const uint32_t row = part * RPT + i;
        float v = 0.0f;
        if (OUT && row < D && col < D) v = from_chunk ? cstate[(size_t)row * D + col] : a.state[state_at + (size_t)row * D + col];
        S[i] = v;
        if (!OUT) dp[i] = 1.0f;
    }
    if (OUT)
        for (uint32_t i = threadIdx.x; i < 4 * PS; i += blockDim.x) us[i] = 0.0f;
    for (uint32_t i = threadIdx.x; i < kWkvTile * 4 * PS; i += blockDim.x) {  // rows beyond D stay zero
        rs[i] = 0.0f;
        ks[i] = 0.0f;
        ws[i] = 0.0f;
    }
    __syncthreads();
    if (OUT)
        for (uint32_t i = threadIdx.x; i < D; i += blockDim.x) us[place(i)] = a.u[h * D + i];

    for (uint32_t t0 = t_begin; t0 < t_end; t0 += kWkvTile) {
        const uint32_t nt = min(kWkvTile, t_end - t0);
        if (p.per_row) {
            for (uint32_t q = threadIdx.x; q < a.rank; q += blockDim.x) lo[q] = tanhf(a.rkvg[(size_t)t0 * a.ld + 4 * HD + q]);
            __syncthreads();
        }
        for (uint32_t i = threadIdx.x; i < nt * D; i += blockDim.x) {
            const uint32_t t = i / D, d = i % D;
            const float* row = a.rkvg + (size_t)(t0 + t) * a.ld + h * D + d;
            if (OUT) rs[t * 4 * PS + place(d)] = row[0];
            ks[t * 4 * PS + place(d)] = row[HD];
            vs[t * D + d] = row[2 * HD];
            float w;
            if (p.per_row) {
                const bf16* w2 = a.w2 + (size_t)(h * D + d) * a.rank_p;
                float acc = 0.0f;
                for (uint32_t q = 0; q < a.rank; ++q) acc = fmaf(__bfloat162float(w2[q]), lo[q], acc);
                w = expf(-expf(acc + a.w0[h * D + d]));
            } else {
                w = a.decay[(size_t)(t0 + t) * HD + h * D + d];
            }
            ws[t * 4 * PS + place(d)] = w;
        }
        __syncthreads();
        if (OUT) {  // bonus of the current token: sum_i r_i u_i k_i
            for (uint32_t t = warp; t < nt; t += n_warps) {
                float b = 0.0f;
                for (uint32_t i = lane; i < 4 * PS; i += 32) b = fmaf(rs[t * 4 * PS + i] * us[i], ks[t * 4 * PS + i], b);
                b = warp_sum_f(b);
                if (lane == 0) bs[t] = b;
            }
            __syncthreads();
        }
        for (uint32_t t = 0; t < nt; ++t) {
            const float v = col < D ? vs[t * D + col] : 0.0f;
            const float4* r4 = reinterpret_cast<const float4*>(rs + t * 4 * PS + part * PS);
            const float4* k4 = reinterpret_cast<const float4*>(ks + t * 4 * PS + part * PS);
            const float4* w4 = reinterpret_cast<const float4*>(ws + t * 4 * PS + part * PS);
            float o = 0.0f;
#pragma unroll
            for (int i = 0; i < RPT / 4; ++i) {
                const float4 k = k4[i], w = w4[i];
                if (OUT) {
                    const float4 r = r4[i];
                    o = fmaf(S[4 * i], r.x, o);
                    o = fmaf(S[4 * i + 1], r.y, o);
                    o = fmaf(S[4 * i + 2], r.z, o);
                    o = fmaf(S[4 * i + 3], r.w, o);
                } else {
                    dp[OUT ? 0 : 4 * i] *= w.x;
                    dp[OUT ? 0 : 4 * i + 1] *= w.y;
                    dp[OUT ? 0 : 4 * i + 2] *= w.z;
                    dp[OUT ? 0 : 4 * i + 3] *= w.w;
                }
                S[4 * i] = fmaf(w.x, S[4 * i], k.x * v);
                S[4 * i + 1] = fmaf(w.y, S[4 * i + 1], k.y * v);
                S[4 * i + 2] = fmaf(w.z, S[4 * i + 2], k.z * v);
                S[4 * i + 3] = fmaf(w.w, S[4 * i + 3], k.w * v);
            }
            if (OUT) {
                o += __shfl_xor_sync(0xFFFFFFFFu, o, 1);
                o += __shfl_xor_sync(0xFFFFFFFFu, o, 2);
                if (part == 0 && col < D) os[t * D + col] = fmaf(bs[t], v, o);
            }
        }
        __syncthreads();
        if (OUT) {
            TA* out = static_cast<TA*>(a.out);
            for (uint32_t t = warp; t < nt; t += n_warps) {
                float ss = 0.0f;
                for (uint32_t d = lane; d < D; d += 32) ss = fmaf(os[t * D + d], os[t * D + d], ss);
                const float inv = 1.0f / sqrtf(warp_sum_f(ss) / (float)D + a.eps);
                const float* g = a.rkvg + (size_t)(t0 + t) * a.ld + 3 * HD + h * D;
                TA* o = out + (size_t)(t0 + t) * a.out_pitch + h * D;
                for (uint32_t d = lane; d < D; d += 32) {
                    const float gv = g[d];
                    o[d] = to_act<TA>(os[t * D + d] * inv * a.norm[h * D + d] * (gv * sigmoid_f(gv)));
                }
                if (h + 1 == a.heads)
                    for (uint32_t c = HD + lane; c < a.out_pitch; c += 32) out[(size_t)(t0 + t) * a.out_pitch + c] = to_act<TA>(0.0f);
            }
            __syncthreads();
        }
    }
    if (OUT) {
        if (p.per_row || chunk + 1 == p.n_chunks) {
#pragma unroll
            for (int i = 0; i < RPT; ++i) {
                const uint32_t row = part * RPT + i;
                if (row < D && col < D) a.state[state_at + (size_t)row * D + col] = S[i];
            }
            if (h == 0 && a.h32 && !p.per_row)  // the token ahead of the next portion
                for (uint32_t i = threadIdx.x; i < a.width; i += blockDim.x)
                    a.prev[(size_t)slot * a.width + i] = a.h32[(size_t)(p.rows - 1) * a.width + i];
        }
    } else {
        float* cdecay = a.chunk + chunk_state * D * D + ((size_t)chunk * a.heads + h) * D;
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const uint32_t row = part * RPT + i;
            if (row < D && col < D) cstate[(size_t)row * D + col] = S[i];
            if (row < D && col == 0) cdecay[row] = dp[OUT ? 0 : i];
        }
    }
}

// Contributions of the chunks -> their starting states, in place: start_0 = the carried state,
// start_(c+1) = decay_c * start_c + contribution_c.
__global__ void __launch_bounds__(256)
wkv_chunk_scan_kernel(const __grid_constant__ WkvParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const WkvArgs& a = p.a;
    const uint32_t D = a.dim, h = blockIdx.y, i = blockIdx.x * 256 + threadIdx.x;
    if (i >= D * D) return;
    const uint32_t slot = (uint32_t)a.slots[0];
    const size_t step = (size_t)a.heads * D * D;
    float* c = a.chunk + (size_t)h * D * D + i;
    const float* dec = a.chunk + (size_t)p.n_chunks * step + (size_t)h * D + i / D;
    float S = a.state[((size_t)slot * a.heads + h) * D * D + i];
    for (uint32_t k = 0; k < p.n_chunks; ++k, c += step, dec += (size_t)a.heads * D) {
        const bool more = k + 1 < p.n_chunks;  // the last chunk's contribution is not needed (and not computed)
        const float own = more ? *c : 0.0f, d = more ? *dec : 0.0f;
        *c = S;
        S = fmaf(d, S, own);
    }
}

int done(cudaError_t e) { return e == cudaSuccess ? ZQ_OK : cuda_fail(e); }

template <int RPT, typename TA>
int wkv_launch(const WkvParams& p, cudaStream_t st) {
    const WkvArgs& a = p.a;
    const uint32_t threads = ((a.dim + 7) / 8) * 32;
    const size_t smem = (kWkvTile * 4 * (RPT + 4) * 3 + 2 * kWkvTile * a.dim + kWkvTile + 4 * (RPT + 4) + a.rank) * sizeof(float);
    if (smem > 200 * 1024) return ZQ_ERR_LIMIT;
    auto read = wkv_kernel<RPT, true, TA>;
    auto sums = wkv_kernel<RPT, false, TA>;
    if (smem > 48 * 1024) {
        ZQ_CUDA(cudaFuncSetAttribute(read, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        ZQ_CUDA(cudaFuncSetAttribute(sums, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    }
    if (!p.per_row && p.n_chunks > 1) {
        int rc = done(launch_pdl(sums, dim3(a.heads, p.n_chunks - 1), dim3(threads), smem, st, p));
        if (rc != ZQ_OK) return rc;
        rc = done(launch_pdl(wkv_chunk_scan_kernel, dim3((a.dim * a.dim + 255) / 256, a.heads), dim3(256), 0, st, p));
        if (rc != ZQ_OK) return rc;
    }
    return done(launch_pdl(read, dim3(a.heads, p.n_chunks), dim3(threads), smem, st, p));
}

template <typename TA>
int wkv_dim(const WkvParams& p, cudaStream_t st) {
    const uint32_t D = p.a.dim;
    if (D <= 32) return wkv_launch<8, TA>(p, st);
    if (D <= 64) return wkv_launch<16, TA>(p, st);
    if (D <= 128) return wkv_launch<32, TA>(p, st);
    return wkv_launch<64, TA>(p, st);
}

}  // namespace

size_t wkv_chunk_floats(uint32_t heads, uint32_t dim, uint32_t max_rows) {
    const size_t n = (max_rows + kWkvChunk - 1) / kWkvChunk;
    return n * heads * ((size_t)dim * dim + dim);
}

int launch_wkv(const WkvArgs& a, uint32_t rows, bool one_sequence, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    if (a.dim == 0 || a.dim > kWkvMaxDim || a.rank == 0) return ZQ_ERR_LIMIT;
    WkvParams p{};
    p.a = a;
    p.rows = rows;
    p.per_row = !one_sequence || rows == 1;
    p.chunk_len = p.per_row ? 1 : kWkvChunk;
    p.n_chunks = (rows + p.chunk_len - 1) / p.chunk_len;
    if (!p.per_row) {
        const size_t smem = (16 * a.rank + 64 * (a.rank + 1)) * sizeof(float);
        if (smem > 200 * 1024) return ZQ_ERR_LIMIT;
        if (smem > 48 * 1024)
            ZQ_CUDA(cudaFuncSetAttribute(wkv_decay_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        const dim3 grid((a.heads * a.dim + 63) / 64, (rows + 15) / 16);
        int rc = done(launch_pdl(wkv_decay_kernel, grid, dim3(256), smem, st, p));
        if (rc != ZQ_OK) return rc;
    }
    return f32 ? wkv_dim<float>(p, st) : wkv_dim<bf16>(p, st);
}

}  // namespace zq
