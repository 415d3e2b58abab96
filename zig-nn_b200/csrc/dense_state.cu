// Recurrences with a matrix state S [dim][vdim] per head, f32, behind gates made from every token:
//   memory   S <- a S + b k v^T, n <- a n + b k with a = exp(f + m - m'), b = exp(i - m'), m' = max(f + m, i);
//            o = S^T q s / (max(|n . q| s, exp(-m')) + 1e-6), s = dim^-1/2
//   delta    S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q
// then every head's o over its root mean square, times a weight and sigmoid(gate).
//
// Value columns are independent of one another. Many tokens of one sequence: in bf16 by chunks on the tensor cores
// (dense_chunk.cuh); in f32, and for a few tokens, a CTA keeps some columns of a head's state in registers (eight threads of
// a warp share a column) and walks the tokens, whose vectors are staged in shared memory ahead of their use. Head norm and
// gate follow in a kernel of their own. One token each of several sequences: a CTA per (sequence, head), with everything
// between the projections in the same kernel.
#include "dense.h"
#include "dense_chunk.cuh"
#include "tile_common.cuh"

namespace zq {
namespace {

constexpr uint32_t kScanTile = 16;    // tokens staged at a time
constexpr uint32_t kScanWarps = 4;    // of four columns each
constexpr uint32_t kStateMaxDim = 512;

__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f(z); }
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }  // bf16 path: 2^-20 or so
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float log_sigmoid_f(float z) { return -softplus_f(-z); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

// ---- many tokens of one sequence ---------------------------------------------------------------------------------
struct ScanParams {
    uint32_t heads, per, dim, vdim, rows;  // per: heads that share a query / key head
    const float *q, *k, *v, *g;            // [rows][...]: head h's vectors at (h / per) * dim, h * vdim, h * dim
    uint32_t q_ld, v_ld, g_ld;
    const float *s0, *s1;                  // memory: z_i, z_f of a head; delta: beta of a head, k . q of a key head
    uint32_t s0_ld, s1_ld;
    const float *i_bias, *f_bias;
    float gate_cap;
    float* S;
    const float *n, *m;
    float *n_end, *m_end;                  // [heads][dim], [heads]: the last token's, stored by the kernel that follows
    const int32_t* slots;
    float* o;                              // [rows][heads * vdim]
};

// Floats of a staged vector: a thread's RPT rows start PS floats after its neighbour's, no bank is met twice.
__host__ __device__ constexpr uint32_t scan_pitch(uint32_t rpt) { return rpt == 4 ? 4 : rpt + 4; }
__host__ __device__ constexpr uint32_t scan_stage_floats(uint32_t rpt, bool delta, uint32_t cols) {
    return kScanTile * ((delta ? 3 : 2) * 8 * scan_pitch(rpt) + cols + 2);
}
inline size_t scan_smem(uint32_t rpt, bool delta, uint32_t cols) {
    return (2 * scan_stage_floats(rpt, delta, cols) + kScanTile * (cols + 2)) * sizeof(float);
}

// The sum over the eight threads of a column of four values; thread `part` gets value ((part & 1) << 1) | (part >> 1 & 1).
__device__ __forceinline__ float sum4_of8(const float (&v)[4], uint32_t part) {
    const bool b0 = part & 1, b1 = part & 2;
    float x = b0 ? v[2] : v[0], y = b0 ? v[3] : v[1];
    x += __shfl_xor_sync(0xFFFFFFFFu, b0 ? v[0] : v[2], 1);
    y += __shfl_xor_sync(0xFFFFFFFFu, b0 ? v[1] : v[3], 1);
    float z = b1 ? y : x;
    z += __shfl_xor_sync(0xFFFFFFFFu, b1 ? x : y, 2);
    return z + __shfl_xor_sync(0xFFFFFFFFu, z, 4);
}

template <int RPT, bool DELTA, bool V4>
__global__ void __launch_bounds__((kScanWarps + 1) * 32)
state_scan_kernel(const __grid_constant__ ScanParams p) {
    constexpr uint32_t PS = scan_pitch(RPT), VP = 8 * PS, TILE = kScanTile;
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    const uint32_t D = p.dim, E = p.vdim, h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t n_warps = (blockDim.x >> 5) - (DELTA ? 0 : 1), C = n_warps * 4, c0 = blockIdx.y * C;
    const bool size_warp = !DELTA && warp == n_warps;  // keeps n instead of columns of S
    const uint32_t part = lane & 7, col = size_warp ? 0 : warp * 4 + (lane >> 3), column = c0 + col;
    const bool real = size_warp || column < E;
    const uint32_t stage = scan_stage_floats(RPT, DELTA, C);
    float* os = sm + 2 * stage;       // [TILE][C]
    float* nq = os + TILE * C;        // [TILE] n . q
    float* em = nq + TILE;            // [TILE] exp(-m)
    auto place = [&](uint32_t i) { return (i / RPT) * PS + i % RPT; };
    for (uint32_t i = tid; i < 2 * stage; i += blockDim.x) sm[i] = 0.0f;  // rows and columns beyond the real ones stay zero
    __syncthreads();
    pdl_wait();

    const uint32_t kv = h / p.per;
    auto fetch = [&](uint32_t b, uint32_t t0) {
        float* base = sm + b * stage;
        const uint32_t nt = min(TILE, p.rows - t0), per = V4 ? D / 4 : D;
        uint32_t t = tid / per, c = tid % per;
        const uint32_t dt = blockDim.x / per, dc = blockDim.x % per;
        while (t < nt) {
            const uint32_t d = V4 ? 4 * c : c;
            float* vec = base + t * VP + place(d);
            const float *q = p.q + (size_t)(t0 + t) * p.q_ld + kv * D + d, *k = p.k + (size_t)(t0 + t) * p.q_ld + kv * D + d;
            const float* g = DELTA ? p.g + (size_t)(t0 + t) * p.g_ld + h * D + d : nullptr;
            if (V4) {
                copy_async16(vec, q);
                copy_async16(vec + TILE * VP, k);
                if (DELTA) copy_async16(vec + 2 * TILE * VP, g);
            } else {
                copy_async4(vec, q);
                copy_async4(vec + TILE * VP, k);
                if (DELTA) copy_async4(vec + 2 * TILE * VP, g);
            }
            t += dt;
            c += dc;
            if (c >= per) {
                c -= per;
                ++t;
            }
        }
        float* vs = base + (DELTA ? 3 : 2) * TILE * VP;
        const uint32_t vc = V4 ? C / 4 : C;
        for (uint32_t i = tid; i < nt * vc; i += blockDim.x) {
            const uint32_t tt = i / vc, cc = (i % vc) * (V4 ? 4 : 1);
            if (c0 + cc >= E) continue;
            const float* v = p.v + (size_t)(t0 + tt) * p.v_ld + h * E + c0 + cc;
            if (V4)
                copy_async16(vs + tt * C + cc, v);
            else
                copy_async4(vs + tt * C + cc, v);
        }
        float* sc = vs + TILE * C;
        for (uint32_t i = tid; i < 2 * nt; i += blockDim.x) {
            const uint32_t tt = i >> 1;
            if (i & 1)
                copy_async4(sc + TILE + tt, p.s1 + (size_t)(t0 + tt) * p.s1_ld + (DELTA ? kv : h));
            else
                copy_async4(sc + tt, p.s0 + (size_t)(t0 + tt) * p.s0_ld + h);
        }
        copy_commit();
    };
    fetch(0, 0);

    const uint32_t slot = (uint32_t)p.slots[0];
    float* state = p.S + ((size_t)slot * p.heads + h) * D * E;
    float S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const uint32_t row = part * RPT + i;
        S[i] = 0.0f;
        if (row < D && real) S[i] = size_warp ? p.n[((size_t)slot * p.heads + h) * D + row] : state[(size_t)row * E + column];
    }
    float m = DELTA ? 0.0f : p.m[(size_t)slot * p.heads + h];
    const float ib = DELTA ? 0.0f : p.i_bias[h], fb = DELTA ? 0.0f : p.f_bias[h];
    const float scale = 1.0f / sqrtf((float)D);

    uint32_t b = 0;
    for (uint32_t t0 = 0; t0 < p.rows; t0 += TILE, b ^= 1) {
        const uint32_t nt = min(TILE, p.rows - t0);
        if (t0 + TILE < p.rows) {
            fetch(b ^ 1, t0 + TILE);
            copy_wait<1>();
        } else {
            copy_wait<0>();
        }
        __syncthreads();
        const float *qs = sm + b * stage, *ks = qs + TILE * VP, *gs = ks + TILE * VP, *vs = qs + (DELTA ? 3 : 2) * TILE * VP,
                    *sc = vs + TILE * C;
        if (DELTA) {
            float4 k[RPT / 4], q[RPT / 4], g[RPT / 4];
            auto get = [&](uint32_t t) {
#pragma unroll
                for (int i = 0; i < RPT / 4; ++i) {
                    k[i] = reinterpret_cast<const float4*>(ks + t * VP + part * PS)[i];
                    q[i] = reinterpret_cast<const float4*>(qs + t * VP + part * PS)[i];
                    g[i] = reinterpret_cast<const float4*>(gs + t * VP + part * PS)[i];
                }
            };
            for (uint32_t t = 0; t < nt; ++t) {
                get(t);
                const float v = vs[t * C + col], beta = sc[t], kq = sc[TILE + t];
                float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f), o = y;
#pragma unroll
                for (int i = 0; i < RPT / 4; ++i) {
                    S[4 * i] *= g[i].x;
                    S[4 * i + 1] *= g[i].y;
                    S[4 * i + 2] *= g[i].z;
                    S[4 * i + 3] *= g[i].w;
                    y.x = fmaf(S[4 * i], k[i].x, y.x);
                    y.y = fmaf(S[4 * i + 1], k[i].y, y.y);
                    y.z = fmaf(S[4 * i + 2], k[i].z, y.z);
                    y.w = fmaf(S[4 * i + 3], k[i].w, y.w);
                    o.x = fmaf(S[4 * i], q[i].x, o.x);
                    o.y = fmaf(S[4 * i + 1], q[i].y, o.y);
                    o.z = fmaf(S[4 * i + 2], q[i].z, o.z);
                    o.w = fmaf(S[4 * i + 3], q[i].w, o.w);
                }
                float ys = (y.x + y.y) + (y.z + y.w), sum = (o.x + o.y) + (o.z + o.w);
#pragma unroll
                for (int off = 1; off <= 4; off <<= 1) {
                    ys += __shfl_xor_sync(0xFFFFFFFFu, ys, off);
                    sum += __shfl_xor_sync(0xFFFFFFFFu, sum, off);
                }
                const float u = beta * (v - ys);
#pragma unroll
                for (int i = 0; i < RPT / 4; ++i) {
                    S[4 * i] = fmaf(k[i].x, u, S[4 * i]);
                    S[4 * i + 1] = fmaf(k[i].y, u, S[4 * i + 1]);
                    S[4 * i + 2] = fmaf(k[i].z, u, S[4 * i + 2]);
                    S[4 * i + 3] = fmaf(k[i].w, u, S[4 * i + 3]);
                }
                if (part == 0) os[t * C + col] = fmaf(u, kq, sum);  // S^T q ahead of the write, and the write's share
            }
        } else {
            // lane t: the gates of the tile's token t; m by a scan over (sum of f, largest i carried along)
            float f = 0.0f, in = -INFINITY;
            if (lane < nt) {
                in = soft_cap(sc[lane] + ib, p.gate_cap);
                f = log_sigmoid_f(soft_cap(sc[TILE + lane] + fb, p.gate_cap));
            }
            float F = f, I = in;
#pragma unroll
            for (int off = 1; off < (int)TILE; off <<= 1) {
                const float Fu = __shfl_up_sync(0xFFFFFFFFu, F, off), Iu = __shfl_up_sync(0xFFFFFFFFu, I, off);
                if (lane >= (uint32_t)off) {
                    I = fmaxf(Iu + F, I);
                    F += Fu;
                }
            }
            const float mt = fmaxf(m + F, I);
            float before = __shfl_up_sync(0xFFFFFFFFu, mt, 1);
            if (lane == 0) before = m;
            const float keep = expf(f + before - mt), add = expf(in - mt);
            if (warp == 0 && lane < nt) em[lane] = expf(-mt);
            m = __shfl_sync(0xFFFFFFFFu, mt, nt - 1);
            for (uint32_t t4 = 0; t4 < nt; t4 += 4) {  // tokens beyond the last: b = 0 and a = 1 leave the state as it is
                float o[4];
#pragma unroll
                for (uint32_t j = 0; j < 4; ++j) {
                    const uint32_t t = t4 + j;
                    float a = __shfl_sync(0xFFFFFFFFu, keep, t), w = __shfl_sync(0xFFFFFFFFu, add, t);
                    if (t >= nt) a = 1.0f, w = 0.0f;
                    const float v = size_warp ? w : w * vs[t * C + col];
                    float4 s = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
                    for (int i = 0; i < RPT / 4; ++i) {
                        const float4 k = reinterpret_cast<const float4*>(ks + t * VP + part * PS)[i],
                                     q = reinterpret_cast<const float4*>(qs + t * VP + part * PS)[i];
                        S[4 * i] = fmaf(a, S[4 * i], k.x * v);
                        S[4 * i + 1] = fmaf(a, S[4 * i + 1], k.y * v);
                        S[4 * i + 2] = fmaf(a, S[4 * i + 2], k.z * v);
                        S[4 * i + 3] = fmaf(a, S[4 * i + 3], k.w * v);
                        s.x = fmaf(S[4 * i], q.x, s.x);
                        s.y = fmaf(S[4 * i + 1], q.y, s.y);
                        s.z = fmaf(S[4 * i + 2], q.z, s.z);
                        s.w = fmaf(S[4 * i + 3], q.w, s.w);
                    }
                    o[j] = (s.x + s.y) + (s.z + s.w);
                }
                const float sum = sum4_of8(o, part);
                const uint32_t t = t4 + (((part & 1) << 1) | ((part >> 1) & 1));
                if (part < 4 && t < nt) {
                    if (!size_warp)
                        os[t * C + col] = sum;
                    else if (lane < 8)
                        nq[t] = sum;
                }
            }
        }
        __syncthreads();  // the read-out is complete, the stage may be filled again
        for (uint32_t i = tid; i < nt * C; i += blockDim.x) {
            const uint32_t t = i / C, c = i % C;
            if (c0 + c >= E) continue;
            float o = os[i];
            if (!DELTA) o = o * scale / (fmaxf(fabsf(nq[t] * scale), em[t]) + 1e-6f);
            p.o[(size_t)(t0 + t) * p.heads * E + h * E + c0 + c] = o;
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const uint32_t row = part * RPT + i;
        if (row >= D || !real) continue;
        if (!size_warp)
            state[(size_t)row * E + column] = S[i];
        else if (blockIdx.y == 0 && lane < 8)
            p.n_end[(size_t)h * D + row] = S[i];
    }
    if (!DELTA && blockIdx.y == 0 && tid == 0) p.m_end[h] = m;
}

// o -> activation rows: over the root mean square of its head, times norm, times sigmoid(gate); a warp per (token, head),
// K values per lane held in registers (0: any number, read twice). nq (chunks, memory): o is first divided by
// max(|nq|, exp(-m)) + 1e-6 of its token and head. What other CTAs of the scan still had to read is stored here: n and m, or
// the inputs that later convolutions need.
struct FinishParams {
    uint32_t heads, vdim, rows, norm_step;  // norm_step: 0 = one weight vector for all heads
    const float *o, *norm, *gate, *nq, *m_of;  // nq, m_of: [rows][heads]
    uint32_t gate_ld;
    float eps;
    void* out;
    uint32_t out_pitch;
    const int32_t *slots, *pos;
    uint32_t dim;
    const float *n_end, *m_end;
    float *n, *m;
    const float* in;         // conv inputs of the rows, pitch ld
    float* ring;
    uint32_t ld, taps, channels;
};

template <int K, typename TA>
__global__ void __launch_bounds__(128)
state_finish_kernel(const __grid_constant__ FinishParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t E = p.vdim, r = blockIdx.x, lane = threadIdx.x & 31, h = blockIdx.y * 4 + (threadIdx.x >> 5);
    if (p.n && r == 0) {
        const uint32_t slot = (uint32_t)p.slots[0], hd = p.heads * p.dim;
        for (uint32_t i = blockIdx.y * blockDim.x + threadIdx.x; i < hd; i += gridDim.y * blockDim.x)
            p.n[(size_t)slot * hd + i] = p.n_end[i];
        for (uint32_t i = blockIdx.y * blockDim.x + threadIdx.x; i < p.heads; i += gridDim.y * blockDim.x)
            p.m[(size_t)slot * p.heads + i] = p.m_end[i];
    }
    if (p.ring && r + p.taps > p.rows) {  // the last taps - 1 rows
        float* to = p.ring + ((size_t)(uint32_t)p.slots[0] * p.taps + (uint32_t)p.pos[r] % p.taps) * p.channels;
        for (uint32_t i = blockIdx.y * blockDim.x + threadIdx.x; i < p.channels; i += gridDim.y * blockDim.x)
            to[i] = p.in[(size_t)r * p.ld + i];
    }
    if (h >= p.heads) return;
    const float* o = p.o + ((size_t)r * p.heads + h) * E;
    const float* g = p.gate + (size_t)r * p.gate_ld + h * E;
    const float* norm = p.norm + h * p.norm_step;
    TA* out = static_cast<TA*>(p.out) + (size_t)r * p.out_pitch;
    if constexpr (K > 0) {
        float x[K], z[K], w[K], by = 1.0f, ss = 0.0f;
#pragma unroll
        for (int j = 0; j < K; ++j) {
            const uint32_t c = lane + 32 * j;
            x[j] = c < E ? o[c] : 0.0f;
            z[j] = c < E ? g[c] : 0.0f;
            w[j] = c < E ? norm[c] : 0.0f;
        }
        if (p.nq) by = 1.0f / (fmaxf(fabsf(p.nq[(size_t)r * p.heads + h]), expf(-p.m_of[(size_t)r * p.heads + h])) + 1e-6f);
#pragma unroll
        for (int j = 0; j < K; ++j) {
            x[j] *= by;
            ss = fmaf(x[j], x[j], ss);
        }
        const float inv = 1.0f / sqrtf(warp_sum_f(ss) / (float)E + p.eps);
#pragma unroll
        for (int j = 0; j < K; ++j)
            if (lane + 32 * j < E) out[h * E + lane + 32 * j] = to_act<TA>(x[j] * inv * w[j] * sigmoid_f(z[j]));
    } else {
        float by = 1.0f, ss = 0.0f;
        if (p.nq) by = 1.0f / (fmaxf(fabsf(p.nq[(size_t)r * p.heads + h]), expf(-p.m_of[(size_t)r * p.heads + h])) + 1e-6f);
        for (uint32_t c = lane; c < E; c += 32) ss = fmaf(o[c] * by, o[c] * by, ss);
        const float inv = by / sqrtf(warp_sum_f(ss) / (float)E + p.eps);
        for (uint32_t c = lane; c < E; c += 32) out[h * E + c] = to_act<TA>(o[c] * inv * norm[c] * sigmoid_f(g[c]));
    }
    if (h == 0)
        for (uint32_t c = p.heads * E + lane; c < p.out_pitch; c += 32) out[c] = to_act<TA>(0.0f);
}

// ---- delta: what comes ahead of the recurrence ---------------------------------------------------------------------
struct DeltaParams {
    DeltaArgs a;
    uint32_t rows, channels;
    // many tokens
    void* low_in;        // [2][max_rows][low.kp] activations
    float* low_out;      // [rows][heads * dim | heads * vdim]; the first part becomes the decays
    float *q, *k, *v, *beta, *kq, *o;
};

// Convolution and silu of one channel of row r; row_first: rows of one sequence that lie ahead of r in `in`.
__device__ __forceinline__ float conv_silu(const DeltaArgs& a, uint32_t channels, uint32_t r, uint32_t ahead, uint32_t pos,
                                           uint32_t slot, uint32_t c) {
    const float* w = a.conv + (size_t)c * a.taps;
    const float* x = a.in + (size_t)r * a.ld + c;
    float acc = 0.0f;
    for (uint32_t back = a.taps - 1; back > 0; --back) {
        float v = 0.0f;
        if (back <= ahead)
            v = x[-(ptrdiff_t)((size_t)back * a.ld)];
        else if (back <= pos)
            v = a.ring[((size_t)slot * a.taps + (pos - back) % a.taps) * channels + c];
        acc = fmaf(w[a.taps - 1 - back], v, acc);
    }
    return silu_f(fmaf(w[a.taps - 1], x[0], acc));
}

__device__ __forceinline__ float channel_decay(float x, float A_log, float dt_bias) { return expf(-expf(A_log) * softplus_f(x + dt_bias)); }

// Inputs of the low-rank products as activation rows.
template <typename TA>
__global__ void __launch_bounds__(128)
delta_low_kernel(const __grid_constant__ DeltaParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const DeltaArgs& a = p.a;
    const uint32_t r = blockIdx.x, kp = a.low.kp;
    const float* x = a.in + (size_t)r * a.ld + p.channels + a.heads;
    TA* to = static_cast<TA*>(p.low_in) + (size_t)r * kp;
    for (uint32_t i = threadIdx.x; i < kp; i += blockDim.x) {
        to[i] = to_act<TA>(i < a.a_rank ? x[i] : 0.0f);
        to[(size_t)a.max_rows * kp + i] = to_act<TA>(i < a.g_rank ? x[a.a_rank + i] : 0.0f);
    }
}

// A warp per (token, item): a key head's q and k, a head's v and beta, a head's decays.
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const __grid_constant__ DeltaParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const DeltaArgs& a = p.a;
    const uint32_t r = blockIdx.x, lane = threadIdx.x & 31, D = a.dim, E = a.vdim, kd = a.kv_heads * D;
    uint32_t item = blockIdx.y * 4 + (threadIdx.x >> 5);
    const uint32_t pos = (uint32_t)a.pos[r], slot = (uint32_t)a.slots[0];
    if (item < a.kv_heads) {
        float *q = p.q + (size_t)r * kd + item * D, *k = p.k + (size_t)r * kd + item * D;
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
        for (uint32_t i = lane; i < D; i += 32) {
            const float x = conv_silu(a, p.channels, r, r, pos, slot, item * D + i);
            const float y = conv_silu(a, p.channels, r, r, pos, slot, kd + item * D + i);
            q[i] = x;
            k[i] = y;
            qq = fmaf(x, x, qq);
            kk = fmaf(y, y, kk);
            qk = fmaf(x, y, qk);
        }
        const float fq = 1.0f / sqrtf(warp_sum_f(qq) + 1e-6f) / sqrtf((float)D), fk = 1.0f / sqrtf(warp_sum_f(kk) + 1e-6f);
        for (uint32_t i = lane; i < D; i += 32) {  // every thread reads back what it wrote
            q[i] *= fq;
            k[i] *= fk;
        }
        qk = warp_sum_f(qk);
        if (lane == 0) p.kq[(size_t)r * a.kv_heads + item] = qk * fq * fk;
        return;
    }
    item -= a.kv_heads;
    if (item < a.heads) {
        for (uint32_t i = lane; i < E; i += 32)
            p.v[(size_t)r * a.heads * E + item * E + i] = conv_silu(a, p.channels, r, r, pos, slot, 2 * kd + item * E + i);
        if (lane == 0) p.beta[(size_t)r * a.heads + item] = sigmoid_f(a.in[(size_t)r * a.ld + p.channels + item]);
        return;
    }
    item -= a.heads;
    if (item >= a.heads) return;
    float* g = p.low_out + (size_t)r * a.heads * (D + E) + item * D;
    for (uint32_t i = lane; i < D; i += 32) g[i] = channel_decay(g[i], a.A_log[item], a.dt_bias[item * D + i]);
}

// The images of the chunks (dense_chunk.cuh): a CTA per (chunk, head), from the projections on.
constexpr uint32_t kConvTokens = 8;  // tokens of a channel that a thread convolves at a time

// Convolution and silu of kConvTokens tokens of one channel, rows t0 on; zeros behind the last row.
template <int TAPS>  // 0: any number
__device__ __forceinline__ void conv_run(const DeltaParams& p, uint32_t ch, uint32_t t0, uint32_t pos0, uint32_t slot,
                                         float (&y)[kConvTokens]) {
    const DeltaArgs& a = p.a;
    if constexpr (TAPS > 0) {
        float x[kConvTokens + TAPS - 1], w[TAPS];
        if constexpr (TAPS == 4) {
            const float4 v = *reinterpret_cast<const float4*>(a.conv + (size_t)ch * 4);
            w[0] = v.x; w[1] = v.y; w[2] = v.z; w[3] = v.w;
        } else {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[j] = a.conv[(size_t)ch * TAPS + j];
        }
        const float* in = a.in + ((ptrdiff_t)t0 - (TAPS - 1)) * (ptrdiff_t)a.ld + ch;
#pragma unroll
        for (int j = 0; j < (int)kConvTokens + TAPS - 1; ++j) {
            const int t = (int)t0 + j - (TAPS - 1);
            x[j] = 0.0f;
            if (t >= 0) {
                if ((uint32_t)t < p.rows) x[j] = in[(size_t)j * a.ld];
            } else if ((int)pos0 + t >= 0) {
                x[j] = a.ring[((size_t)slot * TAPS + (uint32_t)((int)pos0 + t) % TAPS) * p.channels + ch];
            }
        }
#pragma unroll
        for (int t = 0; t < (int)kConvTokens; ++t) {
            float acc = 0.0f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j], x[t + j], acc);
            y[t] = t0 + t < p.rows ? silu_fast(acc) : 0.0f;
        }
    } else {
#pragma unroll
        for (uint32_t t = 0; t < kConvTokens; ++t)
            y[t] = t0 + t < p.rows ? conv_silu(a, p.channels, t0 + t, t0 + t, pos0 + t0 + t, slot, ch) : 0.0f;
    }
}

template <int TAPS>
__global__ void __launch_bounds__(256, 3)
delta_chunk_kernel(const __grid_constant__ DeltaParams p, const __grid_constant__ ChunkParams c) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float beta[kChunk], fq[kChunk], fk[kChunk];
    pdl_launch_dependents();
    pdl_wait();
    const DeltaArgs& a = p.a;
    const uint32_t h = blockIdx.x, chunk = blockIdx.y, t0 = chunk * kChunk, nt = min(kChunk, p.rows - t0);
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t D = a.dim, E = a.vdim, kd = a.kv_heads * D, kv = h / (a.heads / a.kv_heads), dp = c.img.dp;
    const uint32_t slot = (uint32_t)a.slots[0], pos0 = (uint32_t)a.pos[0];
    const ChunkStage s = chunk_stage(sm, dp);
    unsigned char* image = c.images + ((size_t)chunk * a.heads + h) * c.image_bytes;
    if (tid < kChunk) beta[tid] = tid < nt ? sigmoid_f(a.in[(size_t)(t0 + tid) * a.ld + p.channels + h]) : 0.0f;
    {  // decays: a thread keeps to one channel (dp is a power of two)
        const float rate = -expf(a.A_log[h]) * kLog2e;
        const uint32_t width = min(dp, 256u);
        for (uint32_t r = tid & (width - 1); r < dp; r += 256) {
            const float bias = r < D ? a.dt_bias[h * D + r] : 0.0f;
            const float* low = p.low_out + (size_t)t0 * a.heads * (D + E) + h * D + r;
            for (uint32_t t = tid / width; t < kChunk; t += 256 / width) {
                // (2^-150 is 0 already; sums of the logarithms stay small enough for their differences)
                const float x = t < nt && r < D ? fmaxf(rate * softplus_f(low[(size_t)t * a.heads * (D + E)] + bias), -150.0f) : 0.0f;
                s.G[t * s.fp + r] = x;
                s.g[t * s.fp + r] = exp2f(x);
            }
        }
    }
    for (uint32_t i = tid; i < 2 * 2 * dp; i += 256) {  // [q or k][half of the tokens][channel]
        const uint32_t r = i & (dp - 1), which = (i >= dp) + (i >= 2 * dp) + (i >= 3 * dp), at = (which & 1) * kConvTokens;
        float y[kConvTokens];
#pragma unroll
        for (int t = 0; t < (int)kConvTokens; ++t) y[t] = 0.0f;
        if (r < D) conv_run<TAPS>(p, (which & 2 ? kd : 0) + kv * D + r, t0 + at, pos0, slot, y);
        float* to = (which & 2 ? s.k : s.q) + at * s.fp + r;
#pragma unroll
        for (int t = 0; t < (int)kConvTokens; ++t) to[t * s.fp] = y[t];
    }
    __syncthreads();
    const uint32_t columns = c.blocks * kChunkCols;
    for (uint32_t i = tid; i < 2 * columns; i += 256) {
        const bool late = i >= columns;
        const uint32_t r = late ? i - columns : i, at = late ? kConvTokens : 0;
        float y[kConvTokens];
#pragma unroll
        for (int t = 0; t < (int)kConvTokens; ++t) y[t] = 0.0f;
        if (r < E) conv_run<TAPS>(p, 2 * kd + h * E + r, t0 + at, pos0, slot, y);
        float* to = value_at(c, chunk, h, at, r);
#pragma unroll
        for (int t = 0; t < (int)kConvTokens; ++t) to[t * 40] = beta[at + t] * y[t];
    }
    for (uint32_t t = warp; t < kChunk; t += 8) {
        float qq = 0.0f, kk = 0.0f;
        for (uint32_t r = lane; r < D; r += 32) {
            qq = fmaf(s.q[t * s.fp + r], s.q[t * s.fp + r], qq);
            kk = fmaf(s.k[t * s.fp + r], s.k[t * s.fp + r], kk);
        }
        qq = warp_sum_f(qq);
        kk = warp_sum_f(kk);
        if (lane == 0) {
            fq[t] = 1.0f / sqrtf(qq + 1e-6f) / sqrtf((float)D);
            fk[t] = 1.0f / sqrtf(kk + 1e-6f);
        }
    }
    for (uint32_t r = tid; r < dp; r += 256) {
        float sum = 0.0f;
#pragma unroll
        for (uint32_t t = 0; t < kChunk; ++t) {
            sum += s.G[t * s.fp + r];
            s.G[t * s.fp + r] = sum;
        }
        reinterpret_cast<float*>(image + c.img.decay())[r] = exp2f(sum);
    }
    __syncthreads();
    {
        const uint32_t pairs = min(dp / 2, 256u);
        for (uint32_t r = 2 * (tid & (pairs - 1)); r < dp; r += 512) {
            const float2 L = *reinterpret_cast<const float2*>(s.G + (kChunk - 1) * s.fp + r);
            for (uint32_t t = tid / pairs; t < kChunk; t += 256 / pairs) {
                const uint32_t at = t * c.img.pitch + r;
                const float2 q = *reinterpret_cast<const float2*>(s.q + t * s.fp + r),
                             k = *reinterpret_cast<const float2*>(s.k + t * s.fp + r),
                             G = *reinterpret_cast<const float2*>(s.G + t * s.fp + r);
                const float ex = exp2f(G.x), ey = exp2f(G.y), kx = fk[t] * k.x, ky = fk[t] * k.y;
                *reinterpret_cast<uint32_t*>(image + c.img.q() + at * 2) = pack_bf16(fq[t] * q.x * ex, fq[t] * q.y * ey);
                put_split_pair(image, c.img.kd(0), c.img.kd(1), at, kx * exp2f(L.x - G.x), ky * exp2f(L.y - G.y));
                put_split_pair(image, c.img.kg(0), c.img.kg(1), at, beta[t] * kx * ex, beta[t] * ky * ey);
            }
        }
    }
    chunk_squares<true>(s, dp, [&](uint32_t t, uint32_t j, float sa, float sb) {
        put_split(image, c.img.b(0), c.img.b(1), t * kChunkSquare + j, fq[t] * fk[j] * sb);
        s.a[t * 20 + j] = t > j ? -beta[t] * fk[t] * fk[j] * sa : 0.0f;  // with the sign of the substitution below
    });
    __syncthreads();
    if (tid < kChunk) {  // column tid of (1 + A)^-1, the newest term last
        float x[kChunk];
#pragma unroll
        for (int t = 0; t < (int)kChunk; ++t) {
            float acc = (uint32_t)t == tid ? 1.0f : 0.0f;
#pragma unroll
            for (int j = 0; j < t; ++j) acc = fmaf(s.a[t * 20 + j], x[j], acc);
            x[t] = acc;
        }
#pragma unroll
        for (int t = 0; t < (int)kChunk; ++t) put_split(image, c.img.t(0), c.img.t(1), t * kChunkSquare + tid, x[t]);
    }
}

// ---- memory: gates and images of many tokens -------------------------------------------------------------------------
// li, lf [rows][heads]: logarithms of the gates; lm [rows + 1][heads]: the running maximum ahead of every token and at the
// end. A CTA per head; a thread takes consecutive tokens, the maxima meet by a scan over (sum of f, largest i carried along).
__global__ void __launch_bounds__(1024)
memory_gates_kernel(const __grid_constant__ MemoryArgs a, uint32_t rows, float* __restrict__ li, float* __restrict__ lf,
                    float* __restrict__ lm) {
    __shared__ float sum_f[32], top_i[32];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t h = blockIdx.x, H = a.heads, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t per = (rows + blockDim.x - 1) / blockDim.x, t0 = tid * per, t1 = min(rows, t0 + per);
    const float* z = a.in + 2 * (size_t)H * (a.dim + a.vdim) + h;
    const size_t at = (size_t)(uint32_t)a.slots[0] * H + h;
    const float m0 = a.m[at], ib = a.i_bias[h], fb = a.f_bias[h];
    float F = 0.0f, I = -INFINITY;
    for (uint32_t t = t0; t < t1; ++t) {
        const float in = soft_cap(z[(size_t)t * a.ld] + ib, a.gate_cap);
        const float f = log_sigmoid_f(soft_cap(z[(size_t)t * a.ld + H] + fb, a.gate_cap));
        li[(size_t)t * H + h] = in;
        lf[(size_t)t * H + h] = f;
        I = fmaxf(I + f, in);
        F += f;
    }
    auto scan = [&](uint32_t width) {
        for (uint32_t off = 1; off < width; off <<= 1) {
            const float Fu = __shfl_up_sync(0xFFFFFFFFu, F, off), Iu = __shfl_up_sync(0xFFFFFFFFu, I, off);
            if (lane >= off) {
                I = fmaxf(Iu + F, I);
                F += Fu;
            }
        }
    };
    scan(32);
    if (lane == 31) {
        sum_f[warp] = F;
        top_i[warp] = I;
    }
    float Fp = __shfl_up_sync(0xFFFFFFFFu, F, 1), Ip = __shfl_up_sync(0xFFFFFFFFu, I, 1);  // of the warp's threads ahead
    if (lane == 0) Fp = 0.0f, Ip = -INFINITY;
    __syncthreads();
    float m = m0;
    for (uint32_t w = 0; w < warp; ++w) m = fmaxf(m + sum_f[w], top_i[w]);
    m = fmaxf(m + Fp, Ip);
    if (tid == 0) lm[h] = m0;
    for (uint32_t t = t0; t < t1; ++t) {  // every thread reads back what it wrote
        m = fmaxf(m + lf[(size_t)t * H + h], li[(size_t)t * H + h]);
        lm[(size_t)(t + 1) * H + h] = m;
    }
    if (t0 < t1 && t1 == rows) a.m[at] = m;
}

__global__ void __launch_bounds__(256)
memory_chunk_kernel(const __grid_constant__ MemoryArgs a, const __grid_constant__ ChunkParams c, const float* __restrict__ li,
                    const float* __restrict__ lf, const float* __restrict__ lm) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float F[kChunk], I[kChunk], M[kChunk];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t H = a.heads, D = a.dim, E = a.vdim, dp = c.img.dp, h = blockIdx.x, chunk = blockIdx.y, t0 = chunk * kChunk;
    const uint32_t nt = min(kChunk, c.rows - t0), tid = threadIdx.x;
    const ChunkStage s = chunk_stage(sm, dp);
    unsigned char* image = c.images + ((size_t)chunk * H + h) * c.image_bytes;
    for (uint32_t i = tid; i < kChunk * dp; i += 256) {  // (dp is a power of two)
        const uint32_t t = i / dp, r = i & (dp - 1);
        const bool real = t < nt && r < D;
        const float* row = a.in + (size_t)(t0 + t) * a.ld + h * D + r;
        s.q[t * s.fp + r] = real ? row[0] : 0.0f;
        s.k[t * s.fp + r] = real ? row[H * D] : 0.0f;
    }
    const float* v = a.in + (size_t)t0 * a.ld + 2 * H * D + h * E;
    for (uint32_t c0 = 0; c0 < c.blocks * kChunkCols; c0 += 32) {  // column vdim is 1 for every token
        const uint32_t i = c0 + (tid & 31), pair = tid >> 5, t = 2 * pair;
        float2 x = make_float2(0.0f, 0.0f);
        if (i < E) {
            if (t < nt) x.x = v[(size_t)t * a.ld + i];
            if (t + 1 < nt) x.y = v[(size_t)(t + 1) * a.ld + i];
        } else if (i == E) {
            x = make_float2(t < nt ? 1.0f : 0.0f, t + 1 < nt ? 1.0f : 0.0f);
        }
        *value_pair(c, chunk, h, pair, i) = x;
    }
    if (tid < 32) {  // sums of f from the chunk's first token on
        float f = tid < nt ? lf[(size_t)(t0 + tid) * H + h] : 0.0f;
#pragma unroll
        for (int off = 1; off < (int)kChunk; off <<= 1) {
            const float u = __shfl_up_sync(0xFFFFFFFFu, f, off);
            if (tid >= (uint32_t)off) f += u;
        }
        if (tid < kChunk) {
            F[tid] = f;
            I[tid] = tid < nt ? li[(size_t)(t0 + tid) * H + h] : -INFINITY;
            M[tid] = lm[(size_t)(min(t0 + tid, c.rows - 1) + 1) * H + h];
        }
    }
    const float m0 = lm[(size_t)t0 * H + h], scale = 1.0f / sqrtf((float)D);
    __syncthreads();
    const float FL = F[kChunk - 1], ML = M[kChunk - 1];
    for (uint32_t i = tid; i < kChunk * dp / 2; i += 256) {
        const uint32_t t = i / (dp / 2), r = 2 * (i & (dp / 2 - 1)), at = t * c.img.pitch + r;
        const float2 q = *reinterpret_cast<const float2*>(s.q + t * s.fp + r), k = *reinterpret_cast<const float2*>(s.k + t * s.fp + r);
        const float fq = scale * expf(F[t] + m0 - M[t]), fk = expf(FL - F[t] + I[t] - ML);
        *reinterpret_cast<uint32_t*>(image + c.img.q() + at * 2) = pack_bf16(fq * q.x, fq * q.y);
        put_split_pair(image, c.img.kd(0), c.img.kd(1), at, fk * k.x, fk * k.y);
    }
    for (uint32_t r = tid; r < dp; r += blockDim.x) reinterpret_cast<float*>(image + c.img.decay())[r] = expf(FL + m0 - ML);
    chunk_squares<false>(s, dp, [&](uint32_t t, uint32_t j, float, float sb) {
        put_split(image, c.img.b(0), c.img.b(1), t * kChunkSquare + j, j <= t ? scale * expf(F[t] - F[j] + I[j] - M[t]) * sb : 0.0f);
    });
}

// ---- one token of one sequence and head ------------------------------------------------------------------------------
// Threads: CP of them side by side along a row of the state (VEC columns each), RG rows at a time.
struct StepShape {
    uint32_t cp, rg;
};
inline StepShape step_shape(uint32_t vdim, uint32_t vec, uint32_t threads) {
    uint32_t cp = 1;
    while (cp < (vdim + vec - 1) / vec && cp < threads) cp <<= 1;
    return StepShape{cp, threads / cp};
}
template <int VEC>
struct Cols {
    float v[VEC];
};
template <int VEC>
__device__ __forceinline__ Cols<VEC> load_cols(const float* p) {
    Cols<VEC> c;
    if (VEC == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        c.v[0] = x.x; c.v[1 % VEC] = x.y; c.v[2 % VEC] = x.z; c.v[3 % VEC] = x.w;
    } else {
        c.v[0] = *p;
    }
    return c;
}
template <int VEC>
__device__ __forceinline__ void store_cols(float* p, const Cols<VEC>& c) {
    if (VEC == 4)
        *reinterpret_cast<float4*>(p) = make_float4(c.v[0], c.v[1 % VEC], c.v[2 % VEC], c.v[3 % VEC]);
    else
        *p = c.v[0];
}
constexpr int kStepBatch = 8;  // state rows requested together

// Rows d0, d0 + step, ... of columns c ...
template <int VEC>
__device__ __forceinline__ void load_batch(const float* S, uint32_t D, uint32_t E, uint32_t c, uint32_t d0, uint32_t step,
                                           Cols<VEC> (&x)[kStepBatch]) {
#pragma unroll
    for (int j = 0; j < kStepBatch; ++j)
        if (c < E && d0 + j * step < D) x[j] = load_cols<VEC>(S + (size_t)(d0 + j * step) * E + c);
}

// Sum of the row groups' partial columns: red [rg][cp * VEC] -> out[c], c < cp * VEC.
template <int VEC>
__device__ __forceinline__ void meet(float* red, const Cols<VEC>& mine, const StepShape& s, float* out, uint32_t limit) {
    const uint32_t w = s.cp * VEC, cx = threadIdx.x % s.cp, rg = threadIdx.x / s.cp;
#pragma unroll
    for (int e = 0; e < VEC; ++e) red[rg * w + cx * VEC + e] = mine.v[e];
    __syncthreads();
    for (uint32_t c = threadIdx.x; c < w && c < limit; c += blockDim.x) {
        float t = red[c];
        for (uint32_t g = 1; g < s.rg; ++g) t += red[g * w + c];
        out[c] = t;
    }
    __syncthreads();
}

// Head norm and gate of the head's o in shared memory.
template <typename TA>
__device__ __forceinline__ void finish_head(const float* os, const float* gate, const float* norm, uint32_t E, float eps,
                                            TA* row, uint32_t h, uint32_t heads, uint32_t out_pitch, float* red) {
    float ss = 0.0f;
    for (uint32_t c = threadIdx.x; c < E; c += blockDim.x) ss = fmaf(os[c], os[c], ss);
    const float inv = 1.0f / sqrtf(block_sum_f(ss, red) / (float)E + eps);
    for (uint32_t c = threadIdx.x; c < E; c += blockDim.x) row[h * E + c] = to_act<TA>(os[c] * inv * norm[c] * gate[c]);
    if (h + 1 == heads)
        for (uint32_t c = heads * E + threadIdx.x; c < out_pitch; c += blockDim.x) row[c] = to_act<TA>(0.0f);
}

template <int VEC, typename TA>
__global__ void __launch_bounds__(512)
memory_step_kernel(const __grid_constant__ MemoryArgs a, StepShape sh) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red33[33];
    pdl_launch_dependents();
    const uint32_t D = a.dim, E = a.vdim, kd = a.heads * D, vd = a.heads * E, h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x;
    float *qs = sm, *ks = qs + D, *vs = ks + D, *gate = vs + E, *os = gate + E, *red = os + E;
    const float* norm = a.norm + h * E;
    const float ib = a.i_bias[h], fb = a.f_bias[h];
    pdl_wait();
    const float* row = a.in + (size_t)r * a.ld;
    const size_t at = (size_t)(uint32_t)a.slots[r] * a.heads + h;
    float* S = a.S + at * D * E;
    const uint32_t cx = tid % sh.cp, rg = tid / sh.cp;
    Cols<VEC> x[kStepBatch];  // the first rows of the state are requested ahead of everything else
    load_batch<VEC>(S, D, E, cx * VEC, rg, sh.rg, x);
    const float in = soft_cap(row[2 * kd + 2 * vd + h] + ib, a.gate_cap);
    const float f = log_sigmoid_f(soft_cap(row[2 * kd + 2 * vd + a.heads + h] + fb, a.gate_cap));
    const float m0 = a.m[at], m = fmaxf(f + m0, in), keep = expf(f + m0 - m), add = expf(in - m);
    const float scale = 1.0f / sqrtf((float)D);
    float nq = 0.0f;
    for (uint32_t i = tid; i < D; i += blockDim.x) {
        const float q = row[h * D + i] * scale, k = row[kd + h * D + i] * add;  // k with its input gate
        qs[i] = q;
        ks[i] = k;
        const float n = fmaf(keep, a.n[at * D + i], k);
        a.n[at * D + i] = n;
        nq = fmaf(n, q, nq);
    }
    for (uint32_t i = tid; i < E; i += blockDim.x) {
        vs[i] = row[2 * kd + h * E + i];
        gate[i] = sigmoid_f(row[2 * kd + vd + h * E + i]);
    }
    nq = block_sum_f(nq, red33);  // its barriers publish the staged values, and everyone has read m
    if (tid == 0) a.m[at] = m;
    const float size = fmaxf(fabsf(nq), expf(-m)) + 1e-6f;
    for (uint32_t c0 = 0; c0 < E; c0 += sh.cp * VEC) {
        const uint32_t c = c0 + cx * VEC;
        Cols<VEC> o;
#pragma unroll
        for (int e = 0; e < VEC; ++e) o.v[e] = 0.0f;
        if (c < E) {
            float v[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] = vs[c + e];
            for (uint32_t d0 = rg; d0 < D; d0 += kStepBatch * sh.rg) {
                if (c0 + d0 != rg) load_batch<VEC>(S, D, E, c, d0, sh.rg, x);
#pragma unroll
                for (int j = 0; j < kStepBatch; ++j) {
                    const uint32_t d = d0 + j * sh.rg;
                    if (d >= D) break;
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        x[j].v[e] = fmaf(keep, x[j].v[e], ks[d] * v[e]);
                        o.v[e] = fmaf(x[j].v[e], qs[d], o.v[e]);
                    }
                    store_cols<VEC>(S + (size_t)d * E + c, x[j]);
                }
            }
        }
        meet<VEC>(red, o, sh, os + c0, E - c0);
    }
    for (uint32_t c = tid; c < E; c += blockDim.x) os[c] /= size;
    finish_head<TA>(os, gate, norm, E, a.eps, static_cast<TA*>(a.out) + (size_t)r * a.out_pitch, h, a.heads, a.out_pitch, red33);
}

template <int VEC, typename TA>
__global__ void __launch_bounds__(512)
delta_step_kernel(const __grid_constant__ DeltaArgs a, StepShape sh) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red33[33];
    pdl_launch_dependents();
    const uint32_t D = a.dim, E = a.vdim, h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, kp = a.low.kp;
    const uint32_t kd = a.kv_heads * D, vd = a.heads * E, channels = 2 * kd + vd, kv = h / (a.heads / a.kv_heads);
    float *lo = sm, *qs = lo + 2 * kp, *ks = qs + D, *gs = ks + D, *vs = gs + D, *gate = vs + E, *os = gate + E, *ys = os + E,
          *red = ys + E;
    const bf16* low_a = a.low.w + (size_t)h * D * kp;
    const bf16* low_g = a.low.w + ((size_t)a.heads * D + (size_t)h * E) * kp;
    if (tid == 0) prefetch_l2_bulk(low_a, D * kp * 2);
    if (tid == 1) prefetch_l2_bulk(low_g, E * kp * 2);
    const float decay = a.A_log[h];
    pdl_wait();
    const float* row = a.in + (size_t)r * a.ld;
    const uint32_t slot = (uint32_t)a.slots[r], pos = (uint32_t)a.pos[r];
    float* S = a.S + ((size_t)slot * a.heads + h) * D * E;
    const uint32_t cx = tid % sh.cp, rg = tid / sh.cp;
    Cols<VEC> keep[kStepBatch];  // the first rows of the state are requested ahead of everything else
    load_batch<VEC>(S, D, E, cx * VEC, rg, sh.rg, keep);
    const float* low_x = row + channels + a.heads;
    for (uint32_t i = tid; i < kp; i += blockDim.x) {
        lo[i] = i < a.a_rank ? low_x[i] : 0.0f;
        lo[kp + i] = i < a.g_rank ? low_x[a.a_rank + i] : 0.0f;
    }
    float qq = 0.0f, kk = 0.0f;
    float* ring = a.taps > 1 ? a.ring + ((size_t)slot * a.taps + pos % a.taps) * channels : nullptr;
    for (uint32_t i = tid; i < 2 * D + E; i += blockDim.x) {
        const uint32_t c = i < D ? kv * D + i : i < 2 * D ? kd + kv * D + (i - D) : 2 * kd + h * E + (i - 2 * D);
        const float x = conv_silu(a, channels, r, 0, pos, slot, c);
        if (ring) ring[c] = row[c];  // heads that share q and k write the same; nobody reads this place in this step
        if (i < D) {
            qs[i] = x;
            qq = fmaf(x, x, qq);
        } else if (i < 2 * D) {
            ks[i - D] = x;
            kk = fmaf(x, x, kk);
        } else {
            vs[i - 2 * D] = x;
        }
    }
    const float fq = 1.0f / sqrtf(block_sum_f(qq, red33) + 1e-6f) / sqrtf((float)D), fk = 1.0f / sqrtf(block_sum_f(kk, red33) + 1e-6f);
    const float beta = sigmoid_f(row[channels + h]);
    // decays and gates: four neighbouring threads share a row of the low-rank matrix
    const uint32_t sub = tid & 3;
    for (uint32_t base = 0; base < D + E; base += blockDim.x / 4) {
        const uint32_t i = base + (tid >> 2);
        float acc = 0.0f;
        if (i < D + E) {
            const uint4* w = reinterpret_cast<const uint4*>(i < D ? low_a + (size_t)i * kp : low_g + (size_t)(i - D) * kp);
            const float* x = i < D ? lo : lo + kp;
#pragma unroll 4
            for (uint32_t c = sub; c < kp / 8; c += 4) {
                float wf[8];
                unpack8(__ldg(w + c), wf);
                const float4 p = reinterpret_cast<const float4*>(x + 8 * c)[0], q = reinterpret_cast<const float4*>(x + 8 * c)[1];
                acc += (wf[0] * p.x + wf[1] * p.y) + (wf[2] * p.z + wf[3] * p.w) +
                       ((wf[4] * q.x + wf[5] * q.y) + (wf[6] * q.z + wf[7] * q.w));
            }
        }
        acc += __shfl_xor_sync(0xFFFFFFFFu, acc, 1);
        acc += __shfl_xor_sync(0xFFFFFFFFu, acc, 2);
        if (sub == 0 && i < D + E) {
            if (i < D)
                gs[i] = channel_decay(acc, decay, a.dt_bias[h * D + i]);
            else
                gate[i - D] = sigmoid_f(acc);
        }
    }
    float kq = 0.0f;
    for (uint32_t i = tid; i < D; i += blockDim.x) {
        const float q = qs[i] * fq, k = ks[i] * fk;
        qs[i] = q;
        ks[i] = k;
        kq = fmaf(q, k, kq);
    }
    kq = block_sum_f(kq, red33);
    for (uint32_t c0 = 0; c0 < E; c0 += sh.cp * VEC) {
        const uint32_t c = c0 + cx * VEC;
        Cols<VEC> y, o;
#pragma unroll
        for (int e = 0; e < VEC; ++e) y.v[e] = o.v[e] = 0.0f;
        const bool held = D <= kStepBatch * sh.rg;  // one batch: the rows stay in registers
        if (c < E) {
            for (uint32_t d0 = rg; d0 < D; d0 += kStepBatch * sh.rg) {
                if (c0 + d0 != rg) load_batch<VEC>(S, D, E, c, d0, sh.rg, keep);
#pragma unroll
                for (int j = 0; j < kStepBatch; ++j) {
                    const uint32_t d = d0 + j * sh.rg;
                    if (d >= D) break;
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        keep[j].v[e] *= gs[d];
                        y.v[e] = fmaf(keep[j].v[e], ks[d], y.v[e]);
                        o.v[e] = fmaf(keep[j].v[e], qs[d], o.v[e]);
                    }
                }
            }
        }
        meet<VEC>(red, y, sh, ys + c0, E - c0);
        meet<VEC>(red, o, sh, os + c0, E - c0);
        if (c < E) {
            float u[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) u[e] = beta * (vs[c + e] - ys[c + e]);
            for (uint32_t d0 = rg; d0 < D; d0 += kStepBatch * sh.rg) {
                if (!held) {
                    load_batch<VEC>(S, D, E, c, d0, sh.rg, keep);
#pragma unroll
                    for (int j = 0; j < kStepBatch; ++j) {
                        const uint32_t d = d0 + j * sh.rg;
                        if (d >= D) break;
#pragma unroll
                        for (int e = 0; e < VEC; ++e) keep[j].v[e] *= gs[d];
                    }
                }
#pragma unroll
                for (int j = 0; j < kStepBatch; ++j) {
                    const uint32_t d = d0 + j * sh.rg;
                    if (d >= D) break;
#pragma unroll
                    for (int e = 0; e < VEC; ++e) keep[j].v[e] = fmaf(ks[d], u[e], keep[j].v[e]);
                    store_cols<VEC>(S + (size_t)d * E + c, keep[j]);
                }
            }
        }
    }
    for (uint32_t c = tid; c < E; c += blockDim.x) os[c] = fmaf(beta * (vs[c] - ys[c]), kq, os[c]);
    finish_head<TA>(os, gate, a.norm, E, a.eps, static_cast<TA*>(a.out) + (size_t)r * a.out_pitch, h, a.heads, a.out_pitch, red33);
}

// ---- launches ------------------------------------------------------------------------------------------------------
int done(cudaError_t e) { return e == cudaSuccess ? ZQ_OK : cuda_fail(e); }

template <typename K>
int allow_smem(K kern, size_t smem) {
    if (smem > 220 * 1024) return ZQ_ERR_LIMIT;
    if (smem > 48 * 1024) ZQ_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return ZQ_OK;
}

template <int RPT, bool DELTA>
int scan_rpt(const ScanParams& p, bool v4, cudaStream_t st) {
    const uint32_t warps = p.vdim <= 4 * kScanWarps ? (p.vdim + 3) / 4 : kScanWarps, cols = 4 * warps;
    const size_t smem = scan_smem(RPT, DELTA, cols);
    const dim3 grid(p.heads, (p.vdim + cols - 1) / cols), block((warps + (DELTA ? 0 : 1)) * 32);
    auto kern = v4 ? state_scan_kernel<RPT, DELTA, true> : state_scan_kernel<RPT, DELTA, false>;
    const int rc = allow_smem(kern, smem);
    return rc != ZQ_OK ? rc : done(launch_pdl(kern, grid, block, smem, st, p));
}
template <bool DELTA>
int scan(const ScanParams& p, cudaStream_t st) {
    auto aligned = [](const float* q) { return ((uintptr_t)q & 15u) == 0; };
    const bool v4 = p.dim % 4 == 0 && p.vdim % 4 == 0 && p.q_ld % 4 == 0 && p.v_ld % 4 == 0 && (!DELTA || p.g_ld % 4 == 0) &&
                    aligned(p.q) && aligned(p.k) && aligned(p.v) && aligned(p.g);
    if (p.dim <= 32) return scan_rpt<4, DELTA>(p, v4, st);
    if (p.dim <= 64) return scan_rpt<8, DELTA>(p, v4, st);
    if (p.dim <= 128) return scan_rpt<16, DELTA>(p, v4, st);
    if (p.dim <= 256) return scan_rpt<32, DELTA>(p, v4, st);
    return scan_rpt<64, DELTA>(p, v4, st);
}

template <typename TA>
int finish_as(const FinishParams& p, cudaStream_t st) {
    const dim3 grid(p.rows, (p.heads + 3) / 4);
    auto go = [&](auto kern) { return done(launch_pdl(kern, grid, dim3(128), 0, st, p)); };
    if (p.vdim <= 64) return go(state_finish_kernel<2, TA>);
    if (p.vdim <= 128) return go(state_finish_kernel<4, TA>);
    if (p.vdim <= 256) return go(state_finish_kernel<8, TA>);
    return go(state_finish_kernel<0, TA>);
}
int finish(const FinishParams& p, bool f32, cudaStream_t st) { return f32 ? finish_as<float>(p, st) : finish_as<bf16>(p, st); }

uint32_t step_threads(uint32_t dim, uint32_t vdim) {
    const uint32_t n = dim * vdim;
    return n >= 16384 ? 512 : n >= 4096 ? 256 : 128;
}
template <typename Args, typename K>
int step(const Args& a, K vec_f32, K vec_bf16, K one_f32, K one_bf16, size_t floats, uint32_t rows, bool f32, cudaStream_t st) {
    const bool v4 = a.vdim % 4 == 0;
    const uint32_t threads = step_threads(a.dim, a.vdim);
    const StepShape sh = step_shape(a.vdim, v4 ? 4 : 1, threads);
    const size_t smem = (floats + threads * (v4 ? 4 : 1)) * sizeof(float);
    K kern = v4 ? (f32 ? vec_f32 : vec_bf16) : (f32 ? one_f32 : one_bf16);
    const int rc = allow_smem(kern, smem);
    return rc != ZQ_OK ? rc : done(launch_pdl(kern, dim3(a.heads, rows), dim3(threads), smem, st, a, sh));
}

size_t up4(size_t n) { return (n + 3) / 4 * 4; }

}  // namespace

namespace {

// Fewer tokens than this take the token by token form.
constexpr uint32_t kChunkMinRows = 24;

size_t chunk_image_bytes(uint32_t dim, bool delta) { return chunk_image(dim).bytes(delta); }
uint32_t chunk_blocks(uint32_t vdim, bool delta) { return (vdim + (delta ? 0 : 1) + kChunkCols - 1) / kChunkCols; }
size_t chunk_work_floats(uint32_t heads, uint32_t dim, uint32_t vdim, uint32_t max_rows, bool delta) {
    const size_t n = (size_t)((max_rows + kChunk - 1) / kChunk) * heads;
    return n * (chunk_image_bytes(dim, delta) + chunk_blocks(vdim, delta) * kValueBytes) / 4;
}
// The parameters without S and o; images and values of the chunks lie at `work`.
ChunkParams chunk_params(uint32_t heads, uint32_t dim, uint32_t vdim, uint32_t rows, bool delta, const int32_t* slots, float* work) {
    ChunkParams c{};
    c.img = chunk_image(dim);
    c.heads = heads;
    c.dim = dim;
    c.vdim = vdim;
    c.rows = rows;
    c.n_chunks = (rows + kChunk - 1) / kChunk;
    c.blocks = chunk_blocks(vdim, delta);
    c.image_bytes = c.img.bytes(delta);
    c.images = reinterpret_cast<unsigned char*>(work);
    c.values = c.images + (size_t)c.n_chunks * heads * c.image_bytes;
    c.slots = slots;
    return c;
}

}  // namespace

size_t memory_work_floats(uint32_t heads, uint32_t dim, uint32_t vdim, uint32_t max_rows) {
    const size_t chunked = chunk_work_floats(heads, dim, vdim, max_rows, false) + 4 * up4((size_t)(max_rows + 1) * heads);
    return up4((size_t)max_rows * heads * vdim) + up4((size_t)heads * kStateMaxDim) + up4(heads) + chunked;
}

int launch_memory(const MemoryArgs& a, uint32_t rows, bool one_sequence, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    if (a.dim == 0 || a.vdim == 0 || a.dim > kStateMaxDim || a.vdim > 4096) return ZQ_ERR_LIMIT;
    const uint32_t kd = a.heads * a.dim, vd = a.heads * a.vdim;
    if (!one_sequence || rows == 1)
        return step(a, memory_step_kernel<4, float>, memory_step_kernel<4, bf16>, memory_step_kernel<1, float>,
                    memory_step_kernel<1, bf16>, 2 * (size_t)a.dim + 3 * (size_t)a.vdim, rows, f32, st);
    FinishParams f{};
    f.heads = a.heads;
    f.vdim = a.vdim;
    f.rows = rows;
    f.norm_step = a.vdim;
    f.o = a.work;
    f.norm = a.norm;
    f.gate = a.in + 2 * kd + vd;
    f.gate_ld = a.ld;
    f.eps = a.eps;
    f.out = a.out;
    f.out_pitch = a.out_pitch;
    f.slots = a.slots;
    f.dim = a.dim;
    int rc;
    if (!f32 && rows >= kChunkMinRows) {
        const size_t gates = up4((size_t)(rows + 1) * a.heads);
        float *nq = a.work + up4((size_t)rows * vd), *li = nq + gates, *lf = li + gates, *lm = lf + gates;
        ChunkParams c = chunk_params(a.heads, a.dim, a.vdim, rows, false, a.slots, lm + gates);
        c.S = a.S;
        c.n = a.n;
        c.o = a.work;
        c.nq = nq;
        const size_t smem = chunk_stage_floats(c.img.dp) * sizeof(float);
        if ((rc = allow_smem(memory_chunk_kernel, smem)) != ZQ_OK) return rc;
        const uint32_t threads = rows >= 1024 ? 1024 : pad_to(rows, 32);
        if ((rc = done(launch_pdl(memory_gates_kernel, dim3(a.heads), dim3(threads), 0, st, a, rows, li, lf, lm))) != ZQ_OK) return rc;
        rc = done(launch_pdl(memory_chunk_kernel, dim3(a.heads, c.n_chunks), dim3(256), smem, st, a, c, (const float*)li,
                             (const float*)lf, (const float*)lm));
        if (rc != ZQ_OK) return rc;
        if ((rc = chunk_scan_launch(c, false, st)) != ZQ_OK) return rc;
        f.nq = nq;
        f.m_of = lm + a.heads;
        return finish(f, f32, st);
    }
    ScanParams p{};
    p.heads = a.heads;
    p.per = 1;
    p.dim = a.dim;
    p.vdim = a.vdim;
    p.rows = rows;
    p.q = a.in;
    p.k = a.in + kd;
    p.v = a.in + 2 * kd;
    p.q_ld = p.v_ld = p.s0_ld = p.s1_ld = a.ld;
    p.s0 = a.in + 2 * kd + 2 * vd;
    p.s1 = p.s0 + a.heads;
    p.i_bias = a.i_bias;
    p.f_bias = a.f_bias;
    p.gate_cap = a.gate_cap;
    p.S = a.S;
    p.n = a.n;
    p.m = a.m;
    p.slots = a.slots;
    p.o = a.work;
    p.n_end = a.work + up4((size_t)rows * vd);
    p.m_end = p.n_end + up4((size_t)a.heads * kStateMaxDim);
    if ((rc = scan<false>(p, st)) != ZQ_OK) return rc;
    f.n_end = p.n_end;
    f.m_end = p.m_end;
    f.n = a.n;
    f.m = a.m;
    return finish(f, f32, st);
}

size_t delta_work_floats(const DeltaArgs& a, uint32_t max_rows) {
    const size_t R = max_rows, kd = a.kv_heads * a.dim, hd = a.heads * a.dim, vd = a.heads * a.vdim;
    const size_t one = 2 * up4(R * kd) + up4(R * a.heads) + up4(R * a.kv_heads);
    const size_t chunked = chunk_work_floats(a.heads, a.dim, a.vdim, max_rows, true);
    return up4(2 * R * a.low.kp) + up4(R * (hd + vd)) + 2 * up4(R * vd) + (one > chunked ? one : chunked);
}

int launch_delta(const DeltaArgs& a, uint32_t rows, bool one_sequence, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    if (a.dim == 0 || a.vdim == 0 || a.dim > kStateMaxDim || a.vdim > 4096) return ZQ_ERR_LIMIT;
    if (!one_sequence || rows == 1)
        return step(a, delta_step_kernel<4, float>, delta_step_kernel<4, bf16>, delta_step_kernel<1, float>, delta_step_kernel<1, bf16>,
                    2 * (size_t)a.low.kp + 3 * (size_t)a.dim + 4 * (size_t)a.vdim, rows, f32, st);
    if (rows > a.max_rows) return ZQ_ERR_BAD_ARG;
    const uint32_t kd = a.kv_heads * a.dim, hd = a.heads * a.dim, vd = a.heads * a.vdim;
    const size_t R = a.max_rows;
    DeltaParams p{};
    p.a = a;
    p.rows = rows;
    p.channels = 2 * kd + vd;
    p.low_in = a.work;
    p.low_out = a.work + up4(2 * R * a.low.kp);
    p.v = p.low_out + up4(R * (hd + vd));
    p.o = p.v + up4(R * vd);
    p.q = p.o + up4(R * vd);  // from here on, or the images of the chunks
    p.k = p.q + up4(R * kd);
    p.beta = p.k + up4(R * kd);
    p.kq = p.beta + up4(R * a.heads);
    int rc = done(f32 ? launch_pdl(delta_low_kernel<float>, dim3(rows), dim3(128), 0, st, p)
                      : launch_pdl(delta_low_kernel<bf16>, dim3(rows), dim3(128), 0, st, p));
    if (rc != ZQ_OK) return rc;
    LinGroups G{};
    G.n = 2;
    G.g[0] = LinGroup{0, hd, 0, 0};
    G.g[1] = LinGroup{hd, vd, a.max_rows, hd};
    if ((rc = launch_dense_linear(a.low, G, p.low_in, 2 * a.max_rows, rows, p.low_out, hd + vd, f32, st)) != ZQ_OK) return rc;
    FinishParams f{};
    f.heads = a.heads;
    f.vdim = a.vdim;
    f.rows = rows;
    f.o = p.o;
    f.norm = a.norm;
    f.gate = p.low_out + hd;
    f.gate_ld = hd + vd;
    f.eps = a.eps;
    f.out = a.out;
    f.out_pitch = a.out_pitch;
    f.slots = a.slots;
    f.pos = a.pos;
    if (a.taps > 1) {
        f.in = a.in;
        f.ring = a.ring;
        f.ld = a.ld;
        f.taps = a.taps;
        f.channels = p.channels;
    }
    if (!f32 && rows >= kChunkMinRows) {
        ChunkParams c = chunk_params(a.heads, a.dim, a.vdim, rows, true, a.slots, p.q);
        c.S = a.S;
        c.o = p.o;
        const size_t smem = chunk_stage_floats(c.img.dp) * sizeof(float);
        auto kern = a.taps == 4 ? delta_chunk_kernel<4> : delta_chunk_kernel<0>;
        if ((rc = allow_smem(kern, smem)) != ZQ_OK) return rc;
        if ((rc = done(launch_pdl(kern, dim3(a.heads, c.n_chunks), dim3(256), smem, st, p, c))) != ZQ_OK) return rc;
        if ((rc = chunk_scan_launch(c, true, st)) != ZQ_OK) return rc;
        return finish(f, f32, st);
    }
    rc = done(launch_pdl(delta_prepare_kernel, dim3(rows, (a.kv_heads + 2 * a.heads + 3) / 4), dim3(128), 0, st, p));
    if (rc != ZQ_OK) return rc;
    ScanParams s{};
    s.heads = a.heads;
    s.per = a.heads / a.kv_heads;
    s.dim = a.dim;
    s.vdim = a.vdim;
    s.rows = rows;
    s.q = p.q;
    s.k = p.k;
    s.v = p.v;
    s.g = p.low_out;
    s.q_ld = kd;
    s.v_ld = vd;
    s.g_ld = hd + vd;
    s.s0 = p.beta;
    s.s0_ld = a.heads;
    s.s1 = p.kq;
    s.s1_ld = a.kv_heads;
    s.S = a.S;
    s.slots = a.slots;
    s.o = p.o;
    if ((rc = scan<true>(s, st)) != ZQ_OK) return rc;
    return finish(f, f32, st);
}

}  // namespace zq
