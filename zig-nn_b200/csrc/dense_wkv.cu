// The recurrence S_t = diag(w_t) S_(t-1) + k_t v_t^T with read-out o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t, per
// head, state in f32; then every head's o over its root mean square, times a weight and a gate.
//
// A thread holds RPT key rows of one value column of the state; four threads of a warp hold one column, a CTA one
// head. A decode step is one such CTA per (sequence, head), its decays computed there too. Many tokens of one sequence
// are cut into chunks: (1) every chunk's own contribution and decay product from a zero state, all
// chunks at once; (2) the chunks' starting states by a short scan over them; (3) every chunk again with its starting
// state, now with the read-out. Chunk borders are counted from the portion's first token; the state stays f32.
#include "dense.h"
#include "tile_common.cuh"

namespace zq {
namespace {

constexpr uint32_t kWkvTile = 16;    // tokens staged in shared memory at a time
constexpr uint32_t kWkvChunk = 64;   // tokens per chunk
constexpr uint32_t kWkvMaxDim = 256;

struct WkvParams {
    WkvArgs a;
    uint32_t rows, chunk_len, n_chunks;
    bool per_row;          // every row is its own sequence, one token of it
};

// decay[t][c] = exp(-exp(w0[c] + sum_q w2[c][q] tanh(x[t][q]))), x = the w1 columns of rkvg: a CTA takes 64 channels of
// 64 tokens, a thread 16 tokens of one channel.
constexpr uint32_t kDecayTokens = 64;

__global__ void __launch_bounds__(256)
wkv_decay_kernel(const __grid_constant__ WkvParams p) {
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    const WkvArgs& a = p.a;
    const uint32_t HD = a.heads * a.dim, R = a.rank, c0 = blockIdx.x * 64, t0 = blockIdx.y * kDecayTokens;
    float* xs = sm;                       // [R][64 tokens]
    float* ws = sm + kDecayTokens * R;    // [R][65 channels]
    const uint32_t col = threadIdx.x & 63, grp = threadIdx.x >> 6;
    const uint32_t chan = min(c0 + col, HD - 1), tok = min(t0 + col, p.rows - 1);
    for (uint32_t q = grp; q < R; q += 4) ws[q * 65 + col] = __bfloat162float(a.w2[(size_t)chan * a.rank_p + q]);
    pdl_wait();
    for (uint32_t q = grp; q < R; q += 4) xs[q * kDecayTokens + col] = tanhf(a.rkvg[(size_t)tok * a.ld + 4 * HD + q]);
    __syncthreads();
    if (c0 + col >= HD) return;
    float acc[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) acc[i] = 0.0f;
    for (uint32_t q = 0; q < R; ++q) {
        const float w = ws[q * 65 + col];
        const float4* x = reinterpret_cast<const float4*>(xs + q * kDecayTokens + grp * 16);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float4 v = x[i];
            acc[4 * i] = fmaf(w, v.x, acc[4 * i]);
            acc[4 * i + 1] = fmaf(w, v.y, acc[4 * i + 1]);
            acc[4 * i + 2] = fmaf(w, v.z, acc[4 * i + 2]);
            acc[4 * i + 3] = fmaf(w, v.w, acc[4 * i + 3]);
        }
    }
    const float w0 = a.w0[c0 + col];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const uint32_t t = t0 + grp * 16 + i;
        if (t < p.rows) a.decay[(size_t)t * HD + c0 + col] = expf(-expf(acc[i] + w0));
    }
}

// Shared memory of the chunk kernel, in floats: two stages of kWkvTile tokens, the read-out of one.
__host__ __device__ constexpr uint32_t wkv_vec_pitch(uint32_t rpt) { return 4 * (rpt + 4); }
inline size_t wkv_chunk_smem(uint32_t rpt, uint32_t dim) {
    const size_t stage = kWkvTile * (3 * wkv_vec_pitch(rpt) + 2 * (size_t)pad_to(dim, 4));
    return (2 * stage + kWkvTile * (size_t)pad_to(dim, 4) + kWkvTile + wkv_vec_pitch(rpt)) * sizeof(float);
}

// A chunk of one sequence. OUT: read-out and epilogue; otherwise the chunk's contribution from a zero state and its decay
// product. V4: rows of dim floats can be copied 16 bytes at a time.
template <int RPT, bool OUT, bool V4, typename TA>
__global__ void __launch_bounds__(RPT * 16)
wkv_chunk_kernel(const __grid_constant__ WkvParams p) {
    constexpr uint32_t PS = RPT + 4, VP = 4 * PS;  // a thread's rows in the staged vectors have pitch PS: no bank conflicts
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    const WkvArgs& a = p.a;
    const uint32_t D = a.dim, DP = (D + 3) & ~3u, HD = a.heads * D, h = blockIdx.x, chunk = blockIdx.y;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
    const uint32_t part = lane & 3, col = warp * 8 + (lane >> 2);
    const uint32_t stage = kWkvTile * (3 * VP + 2 * DP);
    float* os = sm + 2 * stage;         // [tile][DP]
    float* bs = os + kWkvTile * DP;     // [tile]
    float* us = bs + kWkvTile;          // [VP]
    auto place = [&](uint32_t i) { return (i / RPT) * PS + i % RPT; };
    for (uint32_t i = tid; i < 2 * stage; i += blockDim.x) sm[i] = 0.0f;  // rows beyond D stay zero
    for (uint32_t i = tid; i < VP; i += blockDim.x) us[i] = 0.0f;
    __syncthreads();
    if (OUT)
        for (uint32_t i = tid; i < D; i += blockDim.x) us[place(i)] = a.u[h * D + i];
    pdl_wait();

    const uint32_t t_begin = chunk * p.chunk_len, t_end = min(p.rows, t_begin + p.chunk_len);
    // tokens [t0, t0 + tile) -> stage `b`: r | k | w with the pitch above, then v | g
    auto fetch = [&](uint32_t b, uint32_t t0) {
        float* base = sm + b * stage;
        const uint32_t nt = min(kWkvTile, t_end - t0), per = V4 ? D / 4 : D;
        uint32_t t = tid / per, c = tid % per;
        const uint32_t dt = blockDim.x / per, dc = blockDim.x % per;
        while (t < nt) {
            const uint32_t d = V4 ? 4 * c : c;
            const float* row = a.rkvg + (size_t)(t0 + t) * a.ld + h * D + d;
            const float* dec = a.decay + (size_t)(t0 + t) * HD + h * D + d;
            float* vec = base + t * VP + place(d);
            float* flat = base + kWkvTile * 3 * VP + t * DP + d;
            if (V4) {
                if (OUT) {
                    copy_async16(vec, row);
                    copy_async16(flat + kWkvTile * DP, row + 3 * HD);
                }
                copy_async16(vec + kWkvTile * VP, row + HD);
                copy_async16(vec + 2 * kWkvTile * VP, dec);
                copy_async16(flat, row + 2 * HD);
            } else {
                if (OUT) {
                    copy_async4(vec, row);
                    copy_async4(flat + kWkvTile * DP, row + 3 * HD);
                }
                copy_async4(vec + kWkvTile * VP, row + HD);
                copy_async4(vec + 2 * kWkvTile * VP, dec);
                copy_async4(flat, row + 2 * HD);
            }
            t += dt;
            c += dc;
            if (c >= per) {
                c -= per;
                ++t;
            }
        }
        copy_commit();
    };
    fetch(0, t_begin);

    const uint32_t slot = (uint32_t)a.slots[0];
    const size_t state_at = ((size_t)slot * a.heads + h) * D * D;
    const size_t chunk_state = (size_t)p.n_chunks * a.heads;  // [chunk][head] states, then [chunk][head][D] decays
    float* cstate = a.chunk + ((size_t)chunk * a.heads + h) * D * D;
    const float* from = p.n_chunks > 1 ? cstate : a.state + state_at;
    float S[RPT], dp[OUT ? 1 : RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const uint32_t row = part * RPT + i;
        S[i] = OUT && row < D && col < D ? from[(size_t)row * D + col] : 0.0f;
        if (!OUT) dp[i] = 1.0f;
    }

    uint32_t b = 0;
    for (uint32_t t0 = t_begin; t0 < t_end; t0 += kWkvTile, b ^= 1) {
        const uint32_t nt = min(kWkvTile, t_end - t0);
        if (t0 + kWkvTile < t_end) {
            fetch(b ^ 1, t0 + kWkvTile);
            copy_wait<1>();
        } else {
            copy_wait<0>();
        }
        __syncthreads();
        const float *rs = sm + b * stage, *ks = rs + kWkvTile * VP, *ws = ks + kWkvTile * VP, *vs = ws + kWkvTile * VP,
                    *gs = vs + kWkvTile * DP;
        if (OUT) {  // bonus of the current token: sum_i r_i u_i k_i
            for (uint32_t t = warp; t < nt; t += n_warps) {
                float bonus = 0.0f;
                for (uint32_t i = lane; i < VP; i += 32) bonus = fmaf(rs[t * VP + i] * us[i], ks[t * VP + i], bonus);
                bonus = warp_sum_f(bonus);
                if (lane == 0) bs[t] = bonus;
            }
            __syncthreads();
        }
        for (uint32_t t = 0; t < nt; ++t) {
            const float v = col < D ? vs[t * DP + col] : 0.0f;
            const float4* r4 = reinterpret_cast<const float4*>(rs + t * VP + part * PS);
            const float4* k4 = reinterpret_cast<const float4*>(ks + t * VP + part * PS);
            const float4* w4 = reinterpret_cast<const float4*>(ws + t * VP + part * PS);
            float4 o = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (int i = 0; i < RPT / 4; ++i) {
                const float4 k = k4[i], w = w4[i];
                if (OUT) {
                    const float4 r = r4[i];
                    o.x = fmaf(S[4 * i], r.x, o.x);
                    o.y = fmaf(S[4 * i + 1], r.y, o.y);
                    o.z = fmaf(S[4 * i + 2], r.z, o.z);
                    o.w = fmaf(S[4 * i + 3], r.w, o.w);
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
                float sum = (o.x + o.y) + (o.z + o.w);
                sum += __shfl_xor_sync(0xFFFFFFFFu, sum, 1);
                sum += __shfl_xor_sync(0xFFFFFFFFu, sum, 2);
                if (part == 0 && col < D) os[t * DP + col] = fmaf(bs[t], v, sum);
            }
        }
        __syncthreads();  // the stage may be filled again, the read-out is complete
        if (OUT) {
            TA* out = static_cast<TA*>(a.out);
            for (uint32_t t = warp; t < nt; t += n_warps) {
                float ss = 0.0f;
                for (uint32_t d = lane; d < D; d += 32) ss = fmaf(os[t * DP + d], os[t * DP + d], ss);
                const float inv = 1.0f / sqrtf(warp_sum_f(ss) / (float)D + a.eps);
                TA* o = out + (size_t)(t0 + t) * a.out_pitch + h * D;
                for (uint32_t d = lane; d < D; d += 32) {
                    const float gv = gs[t * DP + d];
                    o[d] = to_act<TA>(os[t * DP + d] * inv * a.norm[h * D + d] * (gv * sigmoid_f(gv)));
                }
                if (h + 1 == a.heads)
                    for (uint32_t c = HD + lane; c < a.out_pitch; c += 32) out[(size_t)(t0 + t) * a.out_pitch + c] = to_act<TA>(0.0f);
            }
            __syncthreads();  // the gates lie in the stage that the next fetch overwrites
        }
    }
    if (OUT) {
        if (chunk + 1 == p.n_chunks) {
#pragma unroll
            for (int i = 0; i < RPT; ++i) {
                const uint32_t row = part * RPT + i;
                if (row < D && col < D) a.state[state_at + (size_t)row * D + col] = S[i];
            }
            if (h == 0 && a.h32)  // the token ahead of the next portion
                for (uint32_t i = tid; i < a.width; i += blockDim.x)
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

// One token of one sequence and head: everything is requested at once, the decay's weights ahead of the wait.
template <int RPT, typename TA>
__global__ void __launch_bounds__(RPT * 16)
wkv_step_kernel(const __grid_constant__ WkvParams p) {
    constexpr uint32_t PS = RPT + 4, VP = 4 * PS;
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[33];
    pdl_launch_dependents();
    const WkvArgs& a = p.a;
    const uint32_t D = a.dim, HD = a.heads * D, h = blockIdx.x, r = blockIdx.y;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t part = lane & 3, col = warp * 8 + (lane >> 2);
    float *rs = sm, *ks = rs + VP, *ws = ks + VP, *vs = ws + VP, *os = vs + D, *lo = os + D;  // lo: [rank_p], 16-byte aligned
    lo = sm + ((3 * VP + 2 * D + 3) & ~3u);
    auto place = [&](uint32_t i) { return (i / RPT) * PS + i % RPT; };
    // four neighbouring threads share a channel's row of W2 (blockDim.x >= 4 * dim)
    const uint32_t chan = tid >> 2, n8 = a.rank_p / 8;
    const uint4* w2 = reinterpret_cast<const uint4*>(a.w2 + (size_t)(h * D + min(chan, D - 1)) * a.rank_p);
    constexpr int AHEAD = 2;
    uint4 wv[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) wv[i] = part + 4 * i < n8 ? __ldg(w2 + part + 4 * i) : make_uint4(0, 0, 0, 0);
    float w0 = 0.0f, u = 0.0f, norm = 0.0f;
    if (chan < D) w0 = a.w0[h * D + chan];
    if (tid < D) {
        u = a.u[h * D + tid];
        norm = a.norm[h * D + tid];
    }
    for (uint32_t i = tid; i < 3 * VP; i += blockDim.x) sm[i] = 0.0f;
    __syncthreads();
    pdl_wait();

    const float* row = a.rkvg + (size_t)r * a.ld;
    const size_t state_at = ((size_t)(uint32_t)a.slots[r] * a.heads + h) * D * D;
    float S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const uint32_t k = part * RPT + i;
        S[i] = k < D && col < D ? a.state[state_at + (size_t)k * D + col] : 0.0f;
    }
    float gate = 0.0f, bonus = 0.0f;
    if (tid < D) {
        const float rv = row[h * D + tid], kv = row[HD + h * D + tid];
        rs[place(tid)] = rv;
        ks[place(tid)] = kv;
        vs[tid] = row[2 * HD + h * D + tid];
        gate = row[3 * HD + h * D + tid];
        bonus = rv * u * kv;
    }
    for (uint32_t q = tid; q < a.rank_p; q += blockDim.x) lo[q] = q < a.rank ? tanhf(row[4 * HD + q]) : 0.0f;
    bonus = block_sum_f(bonus, red);  // its barriers publish the staged values too
    float acc = 0.0f;
    auto dot8 = [&](const uint4& w, uint32_t c) {
        float f[8];
        unpack8(w, f);
        const float4 x = reinterpret_cast<const float4*>(lo + 8 * c)[0], y = reinterpret_cast<const float4*>(lo + 8 * c)[1];
        acc += (f[0] * x.x + f[1] * x.y) + (f[2] * x.z + f[3] * x.w) + ((f[4] * y.x + f[5] * y.y) + (f[6] * y.z + f[7] * y.w));
    };
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
        if (part + 4 * i < n8) dot8(wv[i], part + 4 * i);
    for (uint32_t c = part + 4 * AHEAD; c < n8; c += 4) dot8(__ldg(w2 + c), c);
    acc += __shfl_xor_sync(0xFFFFFFFFu, acc, 1);
    acc += __shfl_xor_sync(0xFFFFFFFFu, acc, 2);
    if (part == 0 && chan < D) ws[place(chan)] = expf(-expf(acc + w0));
    __syncthreads();
    const float v = col < D ? vs[col] : 0.0f;
    float4 o = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < RPT / 4; ++i) {
        const float4 k = reinterpret_cast<const float4*>(ks + part * PS)[i], w = reinterpret_cast<const float4*>(ws + part * PS)[i],
                     q = reinterpret_cast<const float4*>(rs + part * PS)[i];
        o.x = fmaf(S[4 * i], q.x, o.x);
        o.y = fmaf(S[4 * i + 1], q.y, o.y);
        o.z = fmaf(S[4 * i + 2], q.z, o.z);
        o.w = fmaf(S[4 * i + 3], q.w, o.w);
        S[4 * i] = fmaf(w.x, S[4 * i], k.x * v);
        S[4 * i + 1] = fmaf(w.y, S[4 * i + 1], k.y * v);
        S[4 * i + 2] = fmaf(w.z, S[4 * i + 2], k.z * v);
        S[4 * i + 3] = fmaf(w.w, S[4 * i + 3], k.w * v);
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const uint32_t k = part * RPT + i;
        if (k < D && col < D) a.state[state_at + (size_t)k * D + col] = S[i];
    }
    float sum = (o.x + o.y) + (o.z + o.w);
    sum += __shfl_xor_sync(0xFFFFFFFFu, sum, 1);
    sum += __shfl_xor_sync(0xFFFFFFFFu, sum, 2);
    if (part == 0 && col < D) os[col] = fmaf(bonus, v, sum);
    __syncthreads();
    const float ov = tid < D ? os[tid] : 0.0f;
    const float inv = 1.0f / sqrtf(block_sum_f(ov * ov, red) / (float)D + a.eps);
    TA* out = static_cast<TA*>(a.out) + (size_t)r * a.out_pitch;
    if (tid < D) out[h * D + tid] = to_act<TA>(ov * inv * norm * (gate * sigmoid_f(gate)));
    if (h + 1 == a.heads)
        for (uint32_t c = HD + tid; c < a.out_pitch; c += blockDim.x) out[c] = to_act<TA>(0.0f);
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
    constexpr uint32_t B = 8;  // chunks whose values are requested together
    for (uint32_t k0 = 0; k0 < p.n_chunks; k0 += B) {
        float own[B], d[B];
#pragma unroll
        for (uint32_t j = 0; j < B; ++j) {
            const bool more = k0 + j + 1 < p.n_chunks;  // the last chunk's contribution is not needed (and not computed)
            own[j] = more ? c[(k0 + j) * step] : 0.0f;
            d[j] = more ? dec[(size_t)(k0 + j) * a.heads * D] : 0.0f;
        }
#pragma unroll
        for (uint32_t j = 0; j < B; ++j) {
            if (k0 + j < p.n_chunks) c[(k0 + j) * step] = S;
            S = fmaf(d[j], S, own[j]);
        }
    }
}

int done(cudaError_t e) { return e == cudaSuccess ? ZQ_OK : cuda_fail(e); }

template <typename K>
int wkv_smem(K kern, size_t smem) {
    if (smem > 220 * 1024) return ZQ_ERR_LIMIT;
    if (smem > 48 * 1024) ZQ_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return ZQ_OK;
}

template <int RPT, bool V4, typename TA>
int wkv_chunks(const WkvParams& p, dim3 threads, cudaStream_t st) {
    const WkvArgs& a = p.a;
    const size_t smem = wkv_chunk_smem(RPT, a.dim);
    auto read = wkv_chunk_kernel<RPT, true, V4, TA>;
    auto sums = wkv_chunk_kernel<RPT, false, V4, TA>;
    int rc;
    if ((rc = wkv_smem(read, smem)) != ZQ_OK || (rc = wkv_smem(sums, smem)) != ZQ_OK) return rc;
    if (p.n_chunks > 1) {
        rc = done(launch_pdl(sums, dim3(a.heads, p.n_chunks - 1), threads, smem, st, p));
        if (rc != ZQ_OK) return rc;
        rc = done(launch_pdl(wkv_chunk_scan_kernel, dim3((a.dim * a.dim + 255) / 256, a.heads), dim3(256), 0, st, p));
        if (rc != ZQ_OK) return rc;
    }
    return done(launch_pdl(read, dim3(a.heads, p.n_chunks), threads, smem, st, p));
}

template <int RPT, typename TA>
int wkv_launch(const WkvParams& p, cudaStream_t st) {
    const WkvArgs& a = p.a;
    const dim3 threads(((a.dim + 7) / 8) * 32);
    if (p.per_row) {
        const size_t smem = (3 * wkv_vec_pitch(RPT) + 2 * (size_t)a.dim + 4 + a.rank_p) * sizeof(float);
        auto kern = wkv_step_kernel<RPT, TA>;
        const int rc = wkv_smem(kern, smem);
        return rc != ZQ_OK ? rc : done(launch_pdl(kern, dim3(a.heads, p.rows), threads, smem, st, p));
    }
    return a.dim % 4 == 0 && a.ld % 4 == 0 ? wkv_chunks<RPT, true, TA>(p, threads, st) : wkv_chunks<RPT, false, TA>(p, threads, st);
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
        const size_t smem = (kDecayTokens + 65) * (size_t)a.rank * sizeof(float);
        if (smem > 200 * 1024) return ZQ_ERR_LIMIT;
        if (smem > 48 * 1024)
            ZQ_CUDA(cudaFuncSetAttribute(wkv_decay_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        const dim3 grid((a.heads * a.dim + 63) / 64, (rows + kDecayTokens - 1) / kDecayTokens);
        int rc = done(launch_pdl(wkv_decay_kernel, grid, dim3(256), smem, st, p));
        if (rc != ZQ_OK) return rc;
    }
    return f32 ? wkv_dim<float>(p, st) : wkv_dim<bf16>(p, st);
}

}  // namespace zq
