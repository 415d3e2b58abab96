// The chunked form of the matrix-state recurrences (dense_state.cu), for many tokens of one sequence in bf16.
//
// Within a chunk of 16 tokens, with D_t the product of the chunk's decays up to token t (a value per key channel, or one for
// the head), S the state ahead of the chunk, K and Q the chunk's keys and queries:
//   U = T (V' - (K' D) S)      delta: V' = beta v, K' = beta k, T = (1 + A)^-1, A_tj = beta_t sum_r k_t k_j D_t / D_j, j < t
//   U = V                      memory: the input gates are in B and in the last line's keys
//   O = (Q D) S + B U          B_tj = sum_r q_t k_j D_t / D_j, j <= t (memory: relative to the running maximum)
//   S <- D_16 S + (K D_16 / D)^T U
// A first kernel makes, for every chunk and head at once, an image of everything but S, as it will lie in shared memory. The
// scan keeps S in the accumulators of mma.sync: a warp has eight value columns and all key channels, so that warps never
// wait for one another; images come in by bulk copies some chunks ahead. Operands that are accumulators of an earlier product
// are turned within the warp (movmatrix). The products take S, U, B, T and the keys as sums of two bf16 values, so they are
// good to about 2^-16. Waits for copies are bounded, as in gemm_bf16.cu.
#pragma once
#include "dense.h"
#include "tc_common.cuh"
#include "tile_common.cuh"

namespace zq {
namespace {

constexpr uint32_t kChunk = 16;
constexpr uint32_t kChunkCols = 32;     // value columns per CTA, eight per warp
constexpr uint32_t kChunkSquare = 24;   // pitch of a 16 x 16 matrix: no bank is met twice
constexpr uint32_t kValueBytes = kChunk * 40 * 4;
constexpr uint32_t kChunkStages = 8;    // at most

// Where the parts of an image lie, in bytes; dp: key channels, padded to 64, 128, 256 or 512.
struct ChunkImage {
    uint32_t dp, pitch;  // pitch of a row of channels, bf16 values
    __host__ __device__ uint32_t rows() const { return kChunk * pitch * 2; }
    __host__ __device__ uint32_t square() const { return kChunk * kChunkSquare * 2; }
    __host__ __device__ uint32_t q() const { return 0; }
    __host__ __device__ uint32_t kd(uint32_t lo) const { return (1 + lo) * rows(); }
    __host__ __device__ uint32_t b(uint32_t lo) const { return 3 * rows() + lo * square(); }
    __host__ __device__ uint32_t decay() const { return 3 * rows() + 2 * square(); }
    __host__ __device__ uint32_t kg(uint32_t lo) const { return decay() + dp * 4 + lo * rows(); }
    __host__ __device__ uint32_t t(uint32_t lo) const { return kg(2) + lo * square(); }
    __host__ __device__ uint32_t bytes(bool delta) const { return delta ? t(2) : kg(0); }
};
inline ChunkImage chunk_image(uint32_t dim) {
    uint32_t dp = 64;
    while (dp < dim) dp <<= 1;
    return ChunkImage{dp, dp + 8};
}

struct ChunkParams {
    ChunkImage img;
    uint32_t heads, dim, vdim, rows, n_chunks, blocks;  // blocks of kChunkCols columns (memory: column vdim is n, its values are 1)
    uint32_t image_bytes, stages;
    unsigned char* images;  // [chunk][head]
    // [chunk][head][block] of kValueBytes; delta, times beta: [16 tokens][40] floats, memory: [8 pairs of tokens][36] float2
    unsigned char* values;
    float *S, *n;
    const int32_t* slots;
    float *o, *nq;          // [rows][heads * vdim]; memory: [rows][heads] of column vdim
    unsigned int* err;
};
// Place of the values of token t (memory: of tokens 2 pair and 2 pair + 1) in column c.
__device__ __forceinline__ unsigned char* value_block(const ChunkParams& p, uint32_t chunk, uint32_t h, uint32_t c) {
    return p.values + (((size_t)chunk * p.heads + h) * p.blocks + c / kChunkCols) * kValueBytes;
}
__device__ __forceinline__ float* value_at(const ChunkParams& p, uint32_t chunk, uint32_t h, uint32_t t, uint32_t c) {
    return reinterpret_cast<float*>(value_block(p, chunk, h, c)) + t * 40 + c % kChunkCols;
}
__device__ __forceinline__ float2* value_pair(const ChunkParams& p, uint32_t chunk, uint32_t h, uint32_t pair, uint32_t c) {
    return reinterpret_cast<float2*>(value_block(p, chunk, h, c)) + pair * 36 + c % kChunkCols;
}

// x = hi + lo, two bf16 values
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    lo = pack_bf16(a - bf16_lo(hi), b - bf16_hi(hi));
}
__device__ __forceinline__ uint32_t turned(uint32_t x) {  // an 8 x 8 tile of the warp, transposed
    uint32_t y;
    asm("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
    return y;
}
// Accumulators of 16 rows x 8 columns -> the operand that has the 16 rows as its k, in two parts.
__device__ __forceinline__ void split_turned(const float (&x)[4], uint32_t (&hi)[2], uint32_t (&lo)[2]) {
    uint32_t a, b, c, d;
    split2(x[0], x[1], a, b);
    split2(x[2], x[3], c, d);
    hi[0] = turned(a);
    hi[1] = turned(c);
    lo[0] = turned(b);
    lo[1] = turned(d);
}
// d = a b
__device__ __forceinline__ void mma_bf16_first(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
        "{%10,%10,%10,%10};"
        : "=f"(d[0]), "=f"(d[1]), "=f"(d[2]), "=f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1), "f"(0.0f));
}
__device__ __forceinline__ void mma_bf16_or(bool first, float (&d)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
    if (first)
        mma_bf16_first(d, a, b[0], b[1]);
    else
        mma_bf16(d, a, b[0], b[1]);
}

// Four warps of eight columns and one that asks for the images. NT: tiles of 16 channels (dp = 16 NT).
template <int NT, bool DELTA>
__global__ void __launch_bounds__(160)
chunk_scan_kernel(const __grid_constant__ ChunkParams p) {
    extern __shared__ __align__(16) unsigned char chunk_sm[];
    __shared__ __align__(8) unsigned long long bars[2 * kChunkStages];
    __shared__ int abort_flag;
    pdl_launch_dependents();
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, q = lane & 3;
    const uint32_t h = blockIdx.x, E = p.vdim, D = p.dim, HE = p.heads * E;
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(chunk_sm), row_bytes = p.img.pitch * 2;
    const uint32_t bar32 = (uint32_t)__cvta_generic_to_shared(bars);
    auto full = [&](uint32_t s) { return bar32 + s * 8; };
    auto empty = [&](uint32_t s) { return bar32 + (kChunkStages + s) * 8; };
    const uint32_t stage_bytes = p.image_bytes + kValueBytes;
    if (tid == 0) {
        for (uint32_t s = 0; s < p.stages; ++s) {
            mbar_init(full(s), 1);
            mbar_init(empty(s), 4);
        }
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    if (warp == 4) {
        if (lane == 0) {
            asm volatile("fence.proxy.async.global;" ::: "memory");
            uint32_t asked = 0, s = 0, round = 0;
            for (; asked < p.n_chunks; ++asked) {
                if (round > 0 && !mbar_wait(empty(s), (round - 1) & 1u, &abort_flag, p.err)) break;
                const size_t at = (size_t)asked * p.heads + h;
                mbar_expect_tx(full(s), stage_bytes);
                bulk_copy_g2s(base + s * stage_bytes, p.images + at * p.image_bytes, p.image_bytes, full(s));
                bulk_copy_g2s(base + s * stage_bytes + p.image_bytes, p.values + (at * p.blocks + blockIdx.y) * kValueBytes, kValueBytes,
                              full(s));
                mbar_arrive(full(s));
                if (++s == p.stages) {
                    s = 0;
                    ++round;
                }
            }
            if (asked < p.n_chunks)  // copies still in flight land before the CTA may retire
                for (uint32_t back = 1; back <= p.stages && back <= asked; ++back) {
                    const uint32_t c = asked - back;
                    for (uint32_t i = 0; i < kSpinLimit; ++i)
                        if (mbar_try_wait(full(c % p.stages), (c / p.stages) & 1u)) break;
                }
        }
        __syncwarp();
        return;
    }

    const uint32_t col = blockIdx.y * kChunkCols + warp * 8 + 2 * q;  // and col + 1
    const uint32_t slot = (uint32_t)p.slots[0];
    float* state = p.S + ((size_t)slot * p.heads + h) * D * E;
    float* ones = DELTA ? nullptr : p.n + ((size_t)slot * p.heads + h) * D;
    auto at = [&](uint32_t r, uint32_t c) -> float* {
        if (r >= D) return nullptr;
        if (c < E) return state + (size_t)r * E + c;
        return !DELTA && c == E ? ones + r : nullptr;
    };
    float S[NT][4];  // channels 16 i + g (+ 8), columns col, col + 1
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float* s = at(i * 16 + g + (e >> 1) * 8, col + (e & 1));
            S[i][e] = s ? *s : 0.0f;
        }
    const uint32_t row_at = (lane & 15) * row_bytes + (lane >> 4) * 16;                           // 16 tokens x 16 channels
    const uint32_t turn_at = ((lane & 7) + (lane >> 4) * 8) * row_bytes + ((lane >> 3) & 1) * 16;  // 16 channels x 16 tokens
    const uint32_t square_at = (lane & 15) * kChunkSquare * 2 + (lane >> 4) * 16;
    const uint32_t v_at = p.image_bytes + (DELTA ? (g * 40 + warp * 8 + 2 * q) * 4 : (q * 36 + warp * 8 + g) * 8);
    const bool even = (E & 1) == 0;  // pairs of columns can be stored together
    uint32_t stage = 0, phase = 0;
    bool ok = true;
    for (uint32_t c = 0; c < p.n_chunks; ++c) {
        ok = __all_sync(0xFFFFFFFFu, mbar_wait(full(stage), phase, &abort_flag, p.err));
        if (!ok) break;
        const uint32_t img = base + stage * stage_bytes;
        const unsigned char* img_p = chunk_sm + stage * stage_bytes;
        float u[4][4], o[2][4];
        // the image's operands are asked for ahead of their use (up to EARLY tiles of channels of them)
        constexpr int EARLY = NT <= 8 ? NT : 4;
        uint32_t kh[2][4], kl[2][4], qq[2][4];
        auto rows_of = [&](int i) {
            if (DELTA) {
                ldmatrix4(kh[i & 1], img + p.img.kg(0) + row_at + i * 32);
                ldmatrix4(kl[i & 1], img + p.img.kg(1) + row_at + i * 32);
            }
            ldmatrix4(qq[i & 1], img + p.img.q() + row_at + i * 32);
        };
        rows_of(0);
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            uint32_t hi[2], lo[2];
            split_turned(S[i], hi, lo);
            if (i + 1 < NT) rows_of(i + 1);
            if (DELTA) {
                mma_bf16_or(i == 0, u[0], kh[i & 1], hi);
                mma_bf16_or(i == 0, u[1], kh[i & 1], lo);
                mma_bf16_or(i < 2, u[2 + (i & 1)], kl[i & 1], hi);
            }
            mma_bf16_or(i == 0, o[0], qq[i & 1], hi);
            mma_bf16_or(i == 0, o[1], qq[i & 1], lo);
        }
        uint32_t uh[2], ul[2], dh[EARLY][4], dl[EARLY][4], bh[4], bl[4], th[4], tl[4];
        const float2 v0 = *reinterpret_cast<const float2*>(img_p + v_at),
                     v1 = *reinterpret_cast<const float2*>(img_p + v_at + (DELTA ? 8 * 40 * 4 : 4 * 36 * 8));
        if (DELTA) {
            ldmatrix4(th, img + p.img.t(0) + square_at);
            ldmatrix4(tl, img + p.img.t(1) + square_at);
        }
        ldmatrix4(bh, img + p.img.b(0) + square_at);
        ldmatrix4(bl, img + p.img.b(1) + square_at);
#pragma unroll
        for (int i = 0; i < EARLY; ++i) {
            ldmatrix4_trans(dh[i], img + p.img.kd(0) + turn_at + i * 32);
            ldmatrix4_trans(dl[i], img + p.img.kd(1) + turn_at + i * 32);
        }
        const float* decay = reinterpret_cast<const float*>(img_p + p.img.decay()) + g;
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            const float d0 = decay[i * 16], d1 = decay[i * 16 + 8];
            S[i][0] *= d0;
            S[i][1] *= d0;
            S[i][2] *= d1;
            S[i][3] *= d1;
        }
        if (DELTA) {
            const float x[4] = {v0.x - ((u[0][0] + u[1][0]) + (u[2][0] + u[3][0])), v0.y - ((u[0][1] + u[1][1]) + (u[2][1] + u[3][1])),
                                v1.x - ((u[0][2] + u[1][2]) + (u[2][2] + u[3][2])), v1.y - ((u[0][3] + u[1][3]) + (u[2][3] + u[3][3]))};
            uint32_t hi[2], lo[2];
            split_turned(x, hi, lo);
            float y[3][4];
            mma_bf16_first(y[0], th, hi[0], hi[1]);
            mma_bf16_first(y[1], th, lo[0], lo[1]);
            mma_bf16_first(y[2], tl, hi[0], hi[1]);
#pragma unroll
            for (int e = 0; e < 4; ++e) y[0][e] += y[1][e] + y[2][e];
            split_turned(y[0], uh, ul);
        } else {
            split2(v0.x, v0.y, uh[0], ul[0]);
            split2(v1.x, v1.y, uh[1], ul[1]);
        }
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            mma_bf16(S[i], dh[i % EARLY], uh[0], uh[1]);
            mma_bf16(S[i], dh[i % EARLY], ul[0], ul[1]);
            mma_bf16(S[i], dl[i % EARLY], uh[0], uh[1]);
            if (i + EARLY < NT) {
                ldmatrix4_trans(dh[i % EARLY], img + p.img.kd(0) + turn_at + (i + EARLY) * 32);
                ldmatrix4_trans(dl[i % EARLY], img + p.img.kd(1) + turn_at + (i + EARLY) * 32);
            }
        }
        mma_bf16(o[0], bh, uh[0], uh[1]);
        mma_bf16(o[1], bh, ul[0], ul[1]);
        mma_bf16(o[0], bl, uh[0], uh[1]);
        __syncwarp();
        if (lane == 0) mbar_arrive(empty(stage));
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const uint32_t t = c * kChunk + g + half * 8;
            const float x = o[0][half * 2] + o[1][half * 2], y = o[0][half * 2 + 1] + o[1][half * 2 + 1];
            if (t >= p.rows) continue;
            float* to = p.o + (size_t)t * HE + h * E + col;
            if (even && col < E) {
                *reinterpret_cast<float2*>(to) = make_float2(x, y);
            } else {
                if (col < E) to[0] = x;
                if (col + 1 < E) to[1] = y;
            }
            if (!DELTA && (col == E || col + 1 == E)) p.nq[(size_t)t * p.heads + h] = col == E ? x : y;
        }
        if (++stage == p.stages) {
            stage = 0;
            phase ^= 1;
        }
    }
    if (!ok) return;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            float* s = at(i * 16 + g + (e >> 1) * 8, col + (e & 1));
            if (s) *s = S[i][e];
        }
}

// ---- images ---------------------------------------------------------------------------------------------------------
// 16 tokens' vectors in shared memory, pitch dp + 4 floats.
struct ChunkStage {
    float *q, *k, *g, *G;  // G: sums of the logarithms (base 2) of g from the chunk's first token on
    float* a;              // [16][20]
    uint32_t fp;
};
__device__ __forceinline__ ChunkStage chunk_stage(float* sm, uint32_t dp) {
    ChunkStage s;
    s.fp = dp + 4;
    s.q = sm;
    s.k = s.q + kChunk * s.fp;
    s.g = s.k + kChunk * s.fp;
    s.G = s.g + kChunk * s.fp;
    s.a = s.G + kChunk * s.fp;
    return s;
}
inline size_t chunk_stage_floats(uint32_t dp) { return 4 * (size_t)kChunk * (dp + 4) + kChunk * 20; }

// Sums over a warp of 16 values: lane l gets that of value chunk_sum_index(l).
__device__ __forceinline__ uint32_t chunk_sum_index(uint32_t lane) {
    return ((lane & 1) << 3) | ((lane & 2) << 1) | ((lane & 4) >> 1) | ((lane & 8) >> 3);
}
__device__ __forceinline__ float chunk_sum(float (&v)[kChunk], uint32_t lane) {
#pragma unroll
    for (int step = 0; step < 4; ++step) {
        const int n = 8 >> step;  // values kept
        const bool up = (lane >> step) & 1;
#pragma unroll
        for (int i = 0; i < n; ++i) {
            const float keep = up ? v[i + n] : v[i], give = up ? v[i] : v[i + n];
            v[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, give, 1 << step);
        }
    }
    return v[0] + __shfl_xor_sync(0xFFFFFFFFu, v[0], 16);
}

// For every key j and token t, given to put(t, j, a, b): b = sum_r q_t k_j (g_(j+1) .. g_t), DECAY: with the products of g,
// and a likewise of k_t; both 0 where t < j (a also means nothing at t = j). Eight warps, each with a late and an early key.
template <bool DECAY, typename Put>
__device__ __forceinline__ void chunk_squares(const ChunkStage& s, uint32_t dp, Put put) {
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
    for (uint32_t which = 0; which < 2; ++which) {
        const uint32_t j = which ? 15 - warp : warp;
        float a[kChunk], b[kChunk];
#pragma unroll
        for (int t = 0; t < (int)kChunk; ++t) a[t] = b[t] = 0.0f;
        for (uint32_t r = lane * 4; r < dp; r += 128) {
            float4 p = *reinterpret_cast<const float4*>(s.k + j * s.fp + r);
#pragma unroll
            for (int t = 0; t < (int)kChunk; ++t) {
                if ((uint32_t)t < j) continue;  // uniform
                const float4 q = *reinterpret_cast<const float4*>(s.q + t * s.fp + r);
                if (DECAY && (uint32_t)t > j) {
                    const float4 k = *reinterpret_cast<const float4*>(s.k + t * s.fp + r);
                    const float4 g = *reinterpret_cast<const float4*>(s.g + t * s.fp + r);
                    p.x *= g.x; p.y *= g.y; p.z *= g.z; p.w *= g.w;
                    a[t] += (p.x * k.x + p.y * k.y) + (p.z * k.z + p.w * k.w);
                }
                b[t] += (p.x * q.x + p.y * q.y) + (p.z * q.z + p.w * q.w);
            }
        }
        const float sa = DECAY ? chunk_sum(a, lane) : 0.0f, sb = chunk_sum(b, lane);
        if (lane < 16) put(chunk_sum_index(lane), j, sa, sb);
    }
}

__device__ __forceinline__ void put_split(unsigned char* image, uint32_t at_hi, uint32_t at_lo, uint32_t i, float x) {
    const bf16 hi = __float2bfloat16_rn(x);
    reinterpret_cast<bf16*>(image + at_hi)[i] = hi;
    reinterpret_cast<bf16*>(image + at_lo)[i] = __float2bfloat16_rn(x - __bfloat162float(hi));
}
__device__ __forceinline__ void put_split_pair(unsigned char* image, uint32_t at_hi, uint32_t at_lo, uint32_t i, float x, float y) {
    uint32_t hi, lo;
    split2(x, y, hi, lo);
    *reinterpret_cast<uint32_t*>(image + at_hi + i * 2) = hi;
    *reinterpret_cast<uint32_t*>(image + at_lo + i * 2) = lo;
}
inline int chunk_scan_launch(ChunkParams p, bool delta, cudaStream_t st) {
    const uint32_t stage = p.image_bytes + kValueBytes;
    p.stages = 224 * 1024 / stage;
    if (p.stages > kChunkStages) p.stages = kChunkStages;
    if (p.stages < 2) return ZQ_ERR_LIMIT;
    const uint32_t smem = p.stages * stage;
    int rc = device_error_word(&p.err);
    if (rc != ZQ_OK) return rc;
    auto go = [&](auto kern) {
        ZQ_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        const cudaError_t e = launch_pdl(kern, dim3(p.heads, p.blocks), dim3(160), smem, st, p);
        return e == cudaSuccess ? ZQ_OK : cuda_fail(e);
    };
    if (p.img.dp == 64) return delta ? go(chunk_scan_kernel<4, true>) : go(chunk_scan_kernel<4, false>);
    if (p.img.dp == 128) return delta ? go(chunk_scan_kernel<8, true>) : go(chunk_scan_kernel<8, false>);
    if (p.img.dp == 256) return delta ? go(chunk_scan_kernel<16, true>) : go(chunk_scan_kernel<16, false>);
    return delta ? go(chunk_scan_kernel<32, true>) : go(chunk_scan_kernel<32, false>);
}

}  // namespace
}  // namespace zq
