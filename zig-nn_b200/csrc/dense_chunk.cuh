// The chunked form of the matrix-state recurrences (dense_state.cu), for many tokens of one sequence in bf16.
//
// Within a chunk of 16 tokens, with D_t the product of the chunk's decays up to token t (a value per key channel, or one for
// the head), S the state ahead of the chunk, K and Q the chunk's keys and queries:
//   U = T (V' - (K' D) S)      delta: V' = beta v, K' = beta k, T = (1 + A)^-1, A_tj = beta_t sum_r k_t k_j D_t / D_j, j < t
//   U = V                      memory: the input gates are in B and in the last line's keys
//   O = (Q D) S + B U          B_tj = sum_r q_t k_j D_t / D_j, j <= t (memory: relative to the running maximum)
//   S <- D_16 S + (K D_16 / D)^T U
// A first kernel makes, for every chunk and head at once, an image of everything but V and S, as it will lie in shared
// memory. The scan keeps S transposed in the accumulators of mma.sync: a CTA has 32 value columns, four warps share the key
// channels of 16 of them; its products take S, U and the keys as sums of two bf16 values, so they are good to about 2^-16.
#pragma once
#include "dense.h"
#include "tile_common.cuh"

namespace zq {
namespace {

constexpr uint32_t kChunk = 16;
constexpr uint32_t kChunkCols = 32;    // value columns per CTA
constexpr uint32_t kChunkSquare = 24;  // pitch of a 16 x 16 matrix: no bank is met twice

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
    uint32_t heads, dim, vdim, rows, n_chunks, image_bytes, stages;
    unsigned char* images;  // [chunk][head]
    const float* v;         // [rows][..], head h at h * vdim; delta: times beta
    uint32_t v_ld;
    float* S;
    float* n;               // memory: column vdim of the state, its values are 1
    const int32_t* slots;
    float* o;               // [rows][heads * vdim]
    float* nq;              // memory: [rows][heads] of that column
};

// x = hi + lo, two bf16 values
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    lo = pack_bf16(a - bf16_lo(hi), b - bf16_hi(hi));
}
// Accumulators of two neighbouring 8-column tiles -> the operand of 16 columns.
__device__ __forceinline__ void split_tiles(const float (&x)[4], const float (&y)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
    split2(x[0], x[1], hi[0], lo[0]);
    split2(x[2], x[3], hi[1], lo[1]);
    split2(y[0], y[1], hi[2], lo[2]);
    split2(y[2], y[3], hi[3], lo[3]);
}

// NT: 8-channel tiles of a warp (dp = 32 NT).
template <int NT, bool DELTA>
__global__ void __launch_bounds__(256)
chunk_scan_kernel(const __grid_constant__ ChunkParams p) {
    extern __shared__ __align__(16) unsigned char chunk_sm[];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, dq = warp & 3, half = warp >> 2;
    const uint32_t h = blockIdx.x, E = p.vdim, D = p.dim;
    const uint32_t col = blockIdx.y * kChunkCols + half * 16 + (lane >> 2);  // and col + 8
    const uint32_t r0 = dq * NT * 8 + (lane & 3) * 2, tok0 = (lane & 3) * 2;
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(chunk_sm), row_bytes = p.img.pitch * 2;
    // partial products of the four warps of a column block: [2][8 warps][4][32] float4
    float4* parts = reinterpret_cast<float4*>(chunk_sm + p.stages * p.image_bytes);
    const size_t image_step = (size_t)p.heads * p.image_bytes;
    const unsigned char* images = p.images + (size_t)h * p.image_bytes;
    auto fetch = [&](uint32_t c) {
        if (c < p.n_chunks) {
            const uint32_t dst = base + (c % p.stages) * p.image_bytes;
            const unsigned char* src = images + c * image_step;
            for (uint32_t i = tid * 16; i < p.image_bytes; i += 256 * 16) copy16(dst + i, src + i, true);
        }
        copy_commit();
    };
    for (uint32_t c = 0; c + 1 < p.stages; ++c) fetch(c);

    const uint32_t slot = (uint32_t)p.slots[0];
    float* state = p.S + ((size_t)slot * p.heads + h) * D * E;
    float* ones = DELTA ? nullptr : p.n + ((size_t)slot * p.heads + h) * D;
    auto at = [&](uint32_t r, uint32_t c) -> float* {
        if (r >= D) return nullptr;
        if (c < E) return state + (size_t)r * E + c;
        return !DELTA && c == E ? ones + r : nullptr;
    };
    float S[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float* s = at(r0 + n * 8 + (e & 1), col + (e >> 1) * 8);
            S[n][e] = s ? *s : 0.0f;
        }
    // values of a chunk, as accumulators of two 8-token tiles
    auto values = [&](uint32_t c, float (&v)[2][4]) {
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t t = c * kChunk + n * 8 + tok0 + (e & 1), cc = col + (e >> 1) * 8;
                v[n][e] = t >= p.rows ? 0.0f : cc < E ? __ldg(p.v + (size_t)t * p.v_ld + h * E + cc) : !DELTA && cc == E ? 1.0f : 0.0f;
            }
    };
    float v[2][4];
    values(0, v);
    const uint32_t b_row = ((lane >> 4) << 3) + (lane & 7), b_col = ((lane >> 3) & 1) * 16;  // rows as columns of an operand
    const uint32_t t_row = ((lane >> 3) & 1) * 8 + (lane & 7), t_col = (lane >> 4) * 16;     // rows as they are
    for (uint32_t c = 0; c < p.n_chunks; ++c) {
        if (p.stages == 2)
            copy_wait<0>();
        else if (p.stages == 3)
            copy_wait<1>();
        else
            copy_wait<2>();
        __syncthreads();
        fetch(c + p.stages - 1);
        const uint32_t img = base + (c % p.stages) * p.image_bytes;
        float4* mine = parts + ((size_t)(c & 1) * 8 + warp) * 4 * 32 + lane;
        const float4* block = parts + ((size_t)(c & 1) * 8 + half * 4) * 4 * 32 + lane;
        {
            float u[2][2][4], o[2][2][4];  // [hi or lo of S][token tile]
#pragma unroll
            for (int i = 0; i < 16; ++i) u[i >> 3][(i >> 2) & 1][i & 3] = o[i >> 3][(i >> 2) & 1][i & 3] = 0.0f;
#pragma unroll
            for (int k = 0; k < NT / 2; ++k) {
                uint32_t hi[4], lo[4], b[4];
                split_tiles(S[2 * k], S[2 * k + 1], hi, lo);
                const uint32_t off = b_row * row_bytes + b_col + (dq * NT * 8 + k * 16) * 2;
                if (DELTA) {
                    ldmatrix4(b, img + p.img.kg(0) + off);
                    mma_bf16(u[0][0], hi, b[0], b[1]);
                    mma_bf16(u[0][1], hi, b[2], b[3]);
                    mma_bf16(u[1][0], lo, b[0], b[1]);
                    mma_bf16(u[1][1], lo, b[2], b[3]);
                    ldmatrix4(b, img + p.img.kg(1) + off);
                    mma_bf16(u[1][0], hi, b[0], b[1]);
                    mma_bf16(u[1][1], hi, b[2], b[3]);
                }
                ldmatrix4(b, img + p.img.q() + off);
                mma_bf16(o[0][0], hi, b[0], b[1]);
                mma_bf16(o[0][1], hi, b[2], b[3]);
                mma_bf16(o[1][0], lo, b[0], b[1]);
                mma_bf16(o[1][1], lo, b[2], b[3]);
            }
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                if (DELTA)
                    mine[n * 32] = make_float4(u[0][n][0] + u[1][n][0], u[0][n][1] + u[1][n][1], u[0][n][2] + u[1][n][2],
                                               u[0][n][3] + u[1][n][3]);
                mine[(2 + n) * 32] = make_float4(o[0][n][0] + o[1][n][0], o[0][n][1] + o[1][n][1], o[0][n][2] + o[1][n][2],
                                                 o[0][n][3] + o[1][n][3]);
            }
        }
        asm volatile("bar.sync %0, 128;" ::"r"(half + 1) : "memory");
        uint32_t uh[4], ul[4];
        if (DELTA) {
            float x[2][4];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const float4 a = block[n * 32], b = block[(4 + n) * 32], d = block[(8 + n) * 32], e = block[(12 + n) * 32];
                x[n][0] = v[n][0] - ((a.x + b.x) + (d.x + e.x));
                x[n][1] = v[n][1] - ((a.y + b.y) + (d.y + e.y));
                x[n][2] = v[n][2] - ((a.z + b.z) + (d.z + e.z));
                x[n][3] = v[n][3] - ((a.w + b.w) + (d.w + e.w));
            }
            uint32_t hi[4], lo[4], th[4], tl[4];
            split_tiles(x[0], x[1], hi, lo);
            const uint32_t off = b_row * kChunkSquare * 2 + b_col;
            ldmatrix4(th, img + p.img.t(0) + off);
            ldmatrix4(tl, img + p.img.t(1) + off);
            float y[2][4], z[2][4];
#pragma unroll
            for (int i = 0; i < 8; ++i) y[i >> 2][i & 3] = z[i >> 2][i & 3] = 0.0f;
            mma_bf16(y[0], hi, th[0], th[1]);
            mma_bf16(y[1], hi, th[2], th[3]);
            mma_bf16(z[0], lo, th[0], th[1]);
            mma_bf16(z[1], lo, th[2], th[3]);
            mma_bf16(y[0], hi, tl[0], tl[1]);
            mma_bf16(y[1], hi, tl[2], tl[3]);
#pragma unroll
            for (int i = 0; i < 8; ++i) y[i >> 2][i & 3] += z[i >> 2][i & 3];
            split_tiles(y[0], y[1], uh, ul);
        } else {
            split_tiles(v[0], v[1], uh, ul);
        }
        values(c + 1, v);
        // the state: decayed, then the chunk's writes
        const float2* decay = reinterpret_cast<const float2*>(chunk_sm + (c % p.stages) * p.image_bytes + p.img.decay() + r0 * 4);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            const float2 g = decay[n * 4];
            S[n][0] *= g.x;
            S[n][1] *= g.y;
            S[n][2] *= g.x;
            S[n][3] *= g.y;
        }
#pragma unroll
        for (int k = 0; k < NT / 2; ++k) {
            uint32_t b[4], l[4];
            const uint32_t off = t_row * row_bytes + t_col + (dq * NT * 8 + k * 16) * 2;
            ldmatrix4_trans(b, img + p.img.kd(0) + off);
            ldmatrix4_trans(l, img + p.img.kd(1) + off);
            mma_bf16(S[2 * k], uh, b[0], b[1]);
            mma_bf16(S[2 * k + 1], uh, b[2], b[3]);
            mma_bf16(S[2 * k], ul, b[0], b[1]);
            mma_bf16(S[2 * k + 1], ul, b[2], b[3]);
            mma_bf16(S[2 * k], uh, l[0], l[1]);
            mma_bf16(S[2 * k + 1], uh, l[2], l[3]);
        }
        if (dq < 2) {  // read-out of eight tokens
            uint32_t bh[4], bl[4];
            const uint32_t off = b_row * kChunkSquare * 2 + b_col;
            ldmatrix4(bh, img + p.img.b(0) + off);
            ldmatrix4(bl, img + p.img.b(1) + off);
            const uint32_t h0 = dq ? bh[2] : bh[0], h1 = dq ? bh[3] : bh[1], l0 = dq ? bl[2] : bl[0], l1 = dq ? bl[3] : bl[1];
            const float4 a = block[(2 + dq) * 32], b = block[(6 + dq) * 32], d = block[(10 + dq) * 32], e = block[(14 + dq) * 32];
            float o[4] = {(a.x + b.x) + (d.x + e.x), (a.y + b.y) + (d.y + e.y), (a.z + b.z) + (d.z + e.z), (a.w + b.w) + (d.w + e.w)};
            float w[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            mma_bf16(o, uh, h0, h1);
            mma_bf16(w, ul, h0, h1);
            mma_bf16(o, uh, l0, l1);
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const uint32_t t = c * kChunk + dq * 8 + tok0 + (x & 1), cc = col + (x >> 1) * 8;
                if (t >= p.rows) continue;
                if (cc < E)
                    p.o[(size_t)t * p.heads * E + h * E + cc] = o[x] + w[x];
                else if (!DELTA && cc == E)
                    p.nq[(size_t)t * p.heads + h] = o[x] + w[x];
            }
        }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            float* s = at(r0 + n * 8 + (e & 1), col + (e >> 1) * 8);
            if (s) *s = S[n][e];
        }
}

// ---- images ---------------------------------------------------------------------------------------------------------
// 16 tokens' vectors in shared memory, pitch dp + 4 floats.
struct ChunkStage {
    float *q, *k, *g, *G;  // G: sums of the logarithms of g from the chunk's first token on
    float *square_a, *square_b;  // [16][17]
    uint32_t fp;
};
__device__ __forceinline__ ChunkStage chunk_stage(float* sm, uint32_t dp) {
    ChunkStage s;
    s.fp = dp + 4;
    s.q = sm;
    s.k = s.q + kChunk * s.fp;
    s.g = s.k + kChunk * s.fp;
    s.G = s.g + kChunk * s.fp;
    s.square_a = s.G + kChunk * s.fp;
    s.square_b = s.square_a + kChunk * 17;
    return s;
}
inline size_t chunk_stage_floats(uint32_t dp) { return 4 * (size_t)kChunk * (dp + 4) + 2 * kChunk * 17; }

// square_b[t][j] = sum_r q_t k_j (g_(j+1) .. g_t), j <= t; DECAY: with the products of g, and square_a likewise of k_t, j < t.
// Sixteen threads of a warp share a key j (256 threads).
template <bool DECAY>
__device__ __forceinline__ void chunk_squares(const ChunkStage& s, uint32_t dp) {
    const uint32_t j = threadIdx.x >> 4, sub = threadIdx.x & 15, first = (threadIdx.x >> 5) * 2;  // the warp's smaller j
    float sum_a[kChunk], sum_b[kChunk];
#pragma unroll
    for (int t = 0; t < (int)kChunk; ++t) sum_a[t] = sum_b[t] = 0.0f;
    for (uint32_t r = sub * 4; r < dp; r += 64) {
        float4 p = *reinterpret_cast<const float4*>(s.k + j * s.fp + r);
#pragma unroll
        for (int t = 0; t < (int)kChunk; ++t) {
            if ((uint32_t)t < first) continue;
            const float4 q = *reinterpret_cast<const float4*>(s.q + t * s.fp + r);
            if (DECAY) {
                const float4 k = *reinterpret_cast<const float4*>(s.k + t * s.fp + r), g = *reinterpret_cast<const float4*>(s.g + t * s.fp + r);
                if ((uint32_t)t > j) {
                    p.x *= g.x; p.y *= g.y; p.z *= g.z; p.w *= g.w;
                }
                sum_a[t] += (p.x * k.x + p.y * k.y) + (p.z * k.z + p.w * k.w);
            }
            sum_b[t] += (p.x * q.x + p.y * q.y) + (p.z * q.z + p.w * q.w);
        }
    }
#pragma unroll
    for (int t = 0; t < (int)kChunk; ++t) {
        if ((uint32_t)t < first) continue;
#pragma unroll
        for (int off = 1; off <= 8; off <<= 1) {
            if (DECAY) sum_a[t] += __shfl_xor_sync(0xFFFFFFFFu, sum_a[t], off);
            sum_b[t] += __shfl_xor_sync(0xFFFFFFFFu, sum_b[t], off);
        }
        if (sub == 0) {
            if (DECAY) s.square_a[t * 17 + j] = sum_a[t];
            s.square_b[t * 17 + j] = sum_b[t];
        }
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

inline int chunk_scan_launch(ChunkParams p, bool delta, uint32_t columns, cudaStream_t st) {
    const uint32_t parts = 2 * 8 * 4 * 32 * 16;
    p.stages = (220 * 1024 - parts) / p.image_bytes;
    if (p.stages > 4) p.stages = 4;
    if (p.stages < 2) return ZQ_ERR_LIMIT;
    const uint32_t smem = p.stages * p.image_bytes + parts;
    auto go = [&](auto kern) {
        ZQ_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        const cudaError_t e = launch_pdl(kern, dim3(p.heads, (columns + kChunkCols - 1) / kChunkCols), dim3(256), smem, st, p);
        return e == cudaSuccess ? ZQ_OK : cuda_fail(e);
    };
    if (p.img.dp == 64) return delta ? go(chunk_scan_kernel<2, true>) : go(chunk_scan_kernel<2, false>);
    if (p.img.dp == 128) return delta ? go(chunk_scan_kernel<4, true>) : go(chunk_scan_kernel<4, false>);
    if (p.img.dp == 256) return delta ? go(chunk_scan_kernel<8, true>) : go(chunk_scan_kernel<8, false>);
    return delta ? go(chunk_scan_kernel<16, true>) : go(chunk_scan_kernel<16, false>);
}

}  // namespace
}  // namespace zq
