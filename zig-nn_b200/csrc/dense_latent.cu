// Causal attention over a cache of latents: a cache row holds the normed latent c [rank] and a rotated key part [rot] that
// all heads share. Key of head h = [W_uk_h c | key part], value = W_uv_h c, softmax in f32.
//   * decode, and portions of few tokens: W_uk is folded into the query (W_uk_h^T q, as many values as the latent) and W_uv
//     comes behind the weighted sum of latents, so that a cache row serves all heads, as key and as value.
//       latent_query    rows of W_uk over CTAs; one more CTA norms, rotates and writes the token's cache row
//       latent_decode   a CTA per (row, 16 heads, key range): the heads are the rows of the MMAs, the warps share a tile's
//                       keys for the scores and the latent's dimensions for the sum
//       latent_output   ranges brought together, then W_uv
//   * longer portions (bf16): keys and values of every cached token are written out by one tensor-core product and the
//     grouped-query kernels attend (dense_attention.cu).
//   * f32, and latents too long for the tiles: gqa_plain_kernel with one key head between the two foldings.
#include "dense.h"
#include "tile_common.cuh"

namespace zq {
namespace {

constexpr uint32_t kTile = 64;             // keys per tile
constexpr uint32_t kMaxSplits = 64;
constexpr uint32_t kFoldRows = 32;         // longer portions write keys and values out
constexpr uint32_t kMaxRot = 1024;
constexpr uint32_t kQueryRanks = 128;      // latent dimensions per CTA of latent_query
constexpr uint32_t kOutputRows = 32;       // value dimensions per CTA of latent_output

struct LatentParams {
    LatentArgs a;
    float scale2;          // scale * log2(e)
    uint32_t rows, splits, rank_blocks;
    void* q;               // folded [rows][heads][keyp], or [rows][heads][key_pitch]
    uint32_t q_pitch;
    float* part;           // [rows][splits][heads][rank4] sums, then [rows][splits][heads][2] maximum and sum of weights
    uint32_t rank4;        // pitch of a sum
    const void* direct;    // [rows][heads * rank] finished sums instead (act rows of pitch direct_pitch)
    uint32_t direct_pitch;
    // written out: [tokens][heads][q_pitch], [tokens][heads][v_pitch], zeros behind them up to a tile's edge
    bf16 *keys, *values;
    uint32_t tokens, v_pitch;
    int32_t* zero;         // the slot that they count as
};

// Cosines and sines of a row's position, one pair of a vector each.
__device__ __forceinline__ void turns(float2* cs, const float* freq, float pos, uint32_t pairs) {
    for (uint32_t i = threadIdx.x; i < pairs; i += blockDim.x) sincosf(pos * freq[i], &cs[i].y, &cs[i].x);
}
// out[i] = turned x[i] for i < n, zeros up to n_pad
template <typename TA>
__device__ __forceinline__ void rotate_to(const float* x, const float2* cs, uint32_t n, uint32_t n_pad, TA* out, uint32_t tid,
                                          uint32_t step) {
    for (uint32_t i = tid; i < n_pad; i += step) {
        float v = 0.0f;
        if (i < n) {
            const float2 t = cs[i >> 1];
            v = i & 1 ? fmaf(x[i], t.x, x[i - 1] * t.y) : fmaf(x[i], t.x, -(x[i + 1] * t.y));
        }
        out[i] = to_act<TA>(v);
    }
}
// The row's cache entry: normed latent, rotated key part, zeros.
template <typename TA>
__device__ __forceinline__ void write_cache(const LatentArgs& a, uint32_t r, const float2* cs, float* red) {
    const LatentShape& s = a.s;
    const float* x = a.in + (size_t)r * a.ld + s.heads * (s.dim + s.rot);
    const uint32_t pos = (uint32_t)a.pos[r];
    TA* row = static_cast<TA*>(a.cache) + ((size_t)(uint32_t)a.slots[r] * s.ctx + pos) * s.keyp;
    float ss = 0.0f;
    for (uint32_t i = threadIdx.x; i < s.rank; i += blockDim.x) ss = fmaf(x[i], x[i], ss);
    const float inv = 1.0f / sqrtf(block_sum_f(ss, red) / (float)s.rank + a.eps);
    for (uint32_t i = threadIdx.x; i < s.rank; i += blockDim.x) row[i] = to_act<TA>(x[i] * inv * a.norm[i]);
    rotate_to(x + s.rank, cs, s.rot, s.keyp - s.rank, row + s.rank, threadIdx.x, blockDim.x);
}

// CTA (head, block of latent dimensions): W_uk_h^T q; the first block of a head also rotates its query part. The last CTA
// of a row writes the cache.
template <typename TA>
__global__ void __launch_bounds__(128)
latent_query_kernel(const __grid_constant__ LatentParams p) {
    extern __shared__ __align__(16) float qs[];  // [dim]
    __shared__ float red[33], sums[8][kQueryRanks];
    __shared__ float2 cs[kMaxRot / 2];
    pdl_launch_dependents();
    const LatentArgs& a = p.a;
    const LatentShape& s = a.s;
    const uint32_t h = blockIdx.x / p.rank_blocks, block = blockIdx.x % p.rank_blocks, r = blockIdx.y, tid = threadIdx.x;
    if (h >= s.heads) {
        pdl_wait();
        turns(cs, a.freq, (float)(uint32_t)a.pos[r], s.rot / 2);
        __syncthreads();
        write_cache<TA>(a, r, cs, red);
        return;
    }
    // a thread takes eight latent dimensions of every eighth row of W_uk_h
    const uint32_t oct = tid & 15, grp = tid >> 4, at = block * kQueryRanks + oct * 8, kp = a.up.kp;
    const uint4* w = reinterpret_cast<const uint4*>(a.up.w + (size_t)h * s.dim * kp + at);
    const bool in = at < kp;
    constexpr int AHEAD = 4;
    uint4 first[AHEAD];
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
        const uint32_t d = grp + 8 * j;
        first[j] = in && d < s.dim ? __ldg(w + (size_t)d * (kp / 8)) : make_uint4(0, 0, 0, 0);
    }
    pdl_wait();
    const float* q = a.in + (size_t)r * a.ld + h * (s.dim + s.rot);
    for (uint32_t i = tid; i < s.dim; i += blockDim.x) qs[i] = q[i];
    if (block == 0) turns(cs, a.freq, (float)(uint32_t)a.pos[r], s.rot / 2);
    __syncthreads();
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.0f;
    auto add = [&](const uint4& u, uint32_t d) {
        float f[8];
        unpack8(u, f);
        const float x = qs[d];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = fmaf(x, f[e], acc[e]);
    };
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
        if (grp + 8 * j < s.dim) add(first[j], grp + 8 * j);
    if (in) {
#pragma unroll 4
        for (uint32_t d = grp + 8 * AHEAD; d < s.dim; d += 8) add(__ldg(w + (size_t)d * (kp / 8)), d);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) sums[grp][oct * 8 + e] = acc[e];
    __syncthreads();
    TA* out = static_cast<TA*>(p.q) + ((size_t)r * s.heads + h) * p.q_pitch;
    const uint32_t rank = block * kQueryRanks + tid;
    if (rank < s.rank) {
        float t = 0.0f;
#pragma unroll
        for (int g = 0; g < 8; ++g) t += sums[g][tid];
        out[rank] = to_act<TA>(t);
    }
    if (block == 0) rotate_to(q + s.dim, cs, s.rot, p.q_pitch - s.rank, out + s.rank, tid, blockDim.x);
}

// Rows whose keys will be written out: queries [unrotated | rotated] with zeros behind (CTAs y = 0), and the cache (y = 1).
// PAIRS: the parts of a head start at even places.
template <bool PAIRS>
__global__ void __launch_bounds__(256)
latent_rows_kernel(const __grid_constant__ LatentParams p) {
    __shared__ float red[33];
    __shared__ float2 cs[kMaxRot / 2];
    pdl_launch_dependents();
    pdl_wait();
    const LatentArgs& a = p.a;
    const LatentShape& s = a.s;
    const uint32_t r = blockIdx.x, lane = threadIdx.x & 31;
    turns(cs, a.freq, (float)(uint32_t)a.pos[r], s.rot / 2);
    __syncthreads();
    if (blockIdx.y) {
        write_cache<bf16>(a, r, cs, red);
        return;
    }
    for (uint32_t h = threadIdx.x >> 5; h < s.heads; h += blockDim.x >> 5) {
        const float* q = a.in + (size_t)r * a.ld + h * (s.dim + s.rot);
        bf16* out = static_cast<bf16*>(p.q) + ((size_t)r * s.heads + h) * p.q_pitch;
        if (PAIRS) {
#pragma unroll 4
            for (uint32_t i = 2 * lane; i < p.q_pitch; i += 64) {
                float2 x = i < s.dim + s.rot ? *reinterpret_cast<const float2*>(q + i) : make_float2(0.0f, 0.0f);
                if (i >= s.dim && i < s.dim + s.rot) {
                    const float2 t = cs[(i - s.dim) >> 1];
                    x = make_float2(fmaf(x.x, t.x, -(x.y * t.y)), fmaf(x.y, t.x, x.x * t.y));
                }
                *reinterpret_cast<uint32_t*>(out + i) = pack_bf16(x.x, x.y);
            }
        } else {
            for (uint32_t i = lane; i < s.dim; i += 32) out[i] = __float2bfloat16_rn(q[i]);
            rotate_to(q + s.dim, cs, s.rot, p.q_pitch - s.dim, out + s.dim, lane, 32);
        }
    }
    if (r == 0 && threadIdx.x == 0) *p.zero = 0;
}

// The key part of every cached token behind each head's own part of its key, zeros up to the pitch; rows behind the last
// token are zeros (a weight of 0 must meet a finite value).
__global__ void __launch_bounds__(128)
latent_key_part_kernel(const __grid_constant__ LatentParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const LatentArgs& a = p.a;
    const LatentShape& s = a.s;
    const uint32_t t = blockIdx.x, n = p.q_pitch - s.dim;
    const bf16 zero = __float2bfloat16_rn(0.0f);
    bf16* key = p.keys + (size_t)t * s.heads * p.q_pitch;
    if (t >= p.tokens) {
        for (uint32_t i = threadIdx.x; i < s.heads * p.q_pitch; i += blockDim.x) key[i] = zero;
        for (uint32_t i = threadIdx.x; i < s.heads * p.v_pitch; i += blockDim.x) p.values[(size_t)t * s.heads * p.v_pitch + i] = zero;
        return;
    }
    const bf16* from = static_cast<const bf16*>(a.cache) + ((size_t)a.slot0 * s.ctx + t) * s.keyp + s.rank;
    for (uint32_t i = threadIdx.x; i < s.heads * n; i += blockDim.x) {
        const uint32_t h = i / n, c = i % n;
        key[h * p.q_pitch + s.dim + c] = c < s.rot ? from[c] : zero;
    }
}

// Shared memory of the decode kernel: queries, `stages` tiles of keys, weights of a tile.
inline uint32_t decode_smem(uint32_t keyp, uint32_t stages) {
    return (16 + stages * kTile) * (keyp + 8) * 2 + 16 * (kTile + 8) * 2 + 4 * 16 * 4 * 2;
}

// VB: 16-wide blocks of the latent per warp, at most.
template <int VB>
__global__ void __launch_bounds__(128)
latent_decode_kernel(const __grid_constant__ LatentParams p, uint32_t stages) {
    extern __shared__ __align__(16) unsigned char sm[];
    pdl_launch_dependents();
    pdl_wait();
    const LatentArgs& a = p.a;
    const LatentShape& s = a.s;
    const uint32_t split = blockIdx.x, h0 = blockIdx.y * 16, r = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t nh = min(16u, s.heads - h0);
    const uint32_t len = (uint32_t)a.pos[r] + 1;
    const uint32_t per = ((len + p.splits - 1) / p.splits + kTile - 1) / kTile * kTile;
    const uint32_t k_begin = split * per, k_end = min(len, k_begin + per);
    const size_t prow = ((size_t)r * p.splits + split) * s.heads + h0;
    float* part_ml = p.part + (size_t)p.rows * p.splits * s.heads * p.rank4;
    if (k_begin >= k_end) return;  // latent_output counts the ranges that hold keys
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(sm), pitch = (s.keyp + 8) * 2, tile_bytes = kTile * pitch;
    const uint32_t q_at = base, k_at = base + 16 * pitch, p_at = k_at + stages * tile_bytes, ppitch = (kTile + 8) * 2;
    float* tops = reinterpret_cast<float*>(sm + (p_at - base) + 16 * ppitch);  // [4][16], then the sums
    const bf16* cache = static_cast<const bf16*>(a.cache) + (size_t)(uint32_t)a.slots[r] * s.ctx * s.keyp;
    const uint32_t cpr = s.keyp / 8;  // 16-byte pieces of a row
    const uint32_t dr = blockDim.x / cpr, dc = blockDim.x % cpr;
    auto fetch = [&](uint32_t t) {
        const uint32_t dst = k_at + (t % stages) * tile_bytes, k0 = k_begin + t * kTile;
        uint32_t row = tid / cpr, c = tid % cpr;
        while (row < kTile) {
            const bool ok = k0 + row < k_end;
            copy16(dst + row * pitch + c * 16, cache + (size_t)(ok ? k0 + row : k0) * s.keyp + c * 8, ok);
            row += dr;
            c += dc;
            if (c >= cpr) {
                c -= cpr;
                ++row;
            }
        }
    };
    const uint32_t n_tiles = (k_end - k_begin + kTile - 1) / kTile;
    {
        const bf16* q = static_cast<const bf16*>(p.q) + ((size_t)r * s.heads + h0) * s.keyp;
        for (uint32_t i = tid; i < 16 * cpr; i += blockDim.x) {
            const uint32_t row = i / cpr, c = i % cpr;
            copy16(q_at + row * pitch + c * 16, q + (size_t)(row < nh ? row : 0) * s.keyp + c * 8, row < nh);
        }
    }
    for (uint32_t t = 0; t + 1 < stages || t == 0; ++t) {
        if (t < n_tiles) fetch(t);
        copy_commit();
    }
    float o[VB * 2][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int v = 0; v < VB * 2; ++v)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[v][e] = 0.0f;
    const uint32_t blocks = (s.rank + 15) / 16, ks = s.keyp / 16;
    const uint32_t qa = q_at + (lane & 15) * pitch + (lane >> 4) * 16;
    const uint32_t pa = p_at + (lane & 15) * ppitch + (lane >> 4) * 16;
    for (uint32_t t = 0; t < n_tiles; ++t) {
        if (stages > 1) {
            if (t + stages - 1 < n_tiles) fetch(t + stages - 1);
            copy_commit();
            copy_wait<1>();
        } else {
            if (t > 0) {
                fetch(t);
                copy_commit();
            }
            copy_wait<0>();
        }
        __syncthreads();
        const uint32_t tile = k_at + (t % stages) * tile_bytes;
        // scores of this warp's 16 keys: two chains of products
        float sc[2][2][4];
#pragma unroll
        for (int i = 0; i < 16; ++i) sc[i >> 3][(i >> 2) & 1][i & 3] = 0.0f;
        const uint32_t ka = tile + (warp * 16 + ((lane >> 4) << 3) + (lane & 7)) * pitch + ((lane >> 3) & 1) * 16;
        uint32_t kk = 0;
#pragma unroll 2
        for (; kk + 1 < ks; kk += 2) {
            uint32_t qa0[4], qa1[4], b0[4], b1[4];
            ldmatrix4(qa0, qa + kk * 32);
            ldmatrix4(qa1, qa + kk * 32 + 32);
            ldmatrix4(b0, ka + kk * 32);
            ldmatrix4(b1, ka + kk * 32 + 32);
            mma_bf16(sc[0][0], qa0, b0[0], b0[1]);
            mma_bf16(sc[0][1], qa0, b0[2], b0[3]);
            mma_bf16(sc[1][0], qa1, b1[0], b1[1]);
            mma_bf16(sc[1][1], qa1, b1[2], b1[3]);
        }
        if (kk < ks) {
            uint32_t qa0[4], b0[4];
            ldmatrix4(qa0, qa + kk * 32);
            ldmatrix4(b0, ka + kk * 32);
            mma_bf16(sc[0][0], qa0, b0[0], b0[1]);
            mma_bf16(sc[0][1], qa0, b0[2], b0[3]);
        }
        const int lim = (int)(k_end - k_begin) - (int)(t * kTile + warp * 16);  // keys of the 16 that exist
        float x[2][4], mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int col = n * 8 + (lane & 3) * 2 + (e & 1);
                x[n][e] = col < lim ? (sc[0][n][e] + sc[1][n][e]) * p.scale2 : -INFINITY;
                if (e < 2)
                    mx0 = fmaxf(mx0, x[n][e]);
                else
                    mx1 = fmaxf(mx1, x[n][e]);
            }
#pragma unroll
        for (int off = 1; off <= 2; off <<= 1) {
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xFFFFFFFFu, mx0, off));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xFFFFFFFFu, mx1, off));
        }
        const uint32_t r0 = lane >> 2, r1 = r0 + 8;
        if ((lane & 3) == 0) {
            tops[warp * 16 + r0] = mx0;
            tops[warp * 16 + r1] = mx1;
        }
        __syncthreads();
        float n0 = m[0], n1 = m[1];
#pragma unroll
        for (uint32_t w = 0; w < 4; ++w) {
            n0 = fmaxf(n0, tops[w * 16 + r0]);
            n1 = fmaxf(n1, tops[w * 16 + r1]);
        }
        // (the tile's first key exists, so the maxima are finite)
        const float f0 = exp2f(m[0] - n0), f1 = exp2f(m[1] - n1);
        m[0] = n0;
        m[1] = n1;
        float a0 = 0.0f, a1 = 0.0f;
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const __nv_bfloat162 top = __floats2bfloat162_rn(exp2f(x[n][0] - n0), exp2f(x[n][1] - n0));
            const __nv_bfloat162 bot = __floats2bfloat162_rn(exp2f(x[n][2] - n1), exp2f(x[n][3] - n1));
            a0 += __low2float(top) + __high2float(top);
            a1 += __low2float(bot) + __high2float(bot);
            unsigned char* at = sm + (p_at - base) + (warp * 16 + n * 8 + (lane & 3) * 2) * 2;
            *reinterpret_cast<__nv_bfloat162*>(at + r0 * ppitch) = top;
            *reinterpret_cast<__nv_bfloat162*>(at + r1 * ppitch) = bot;
        }
        l[0] = l[0] * f0 + a0;  // this lane's share of the sums
        l[1] = l[1] * f1 + a1;
        __syncthreads();
#pragma unroll
        for (int v = 0; v < VB * 2; ++v) {
            o[v][0] *= f0; o[v][1] *= f0; o[v][2] *= f1; o[v][3] *= f1;
        }
        uint32_t pw[4][4];
#pragma unroll
        for (int n = 0; n < 4; ++n) ldmatrix4(pw[n], pa + n * 32);
        const uint32_t va = tile + (((lane >> 3) & 1) * 8 + (lane & 7)) * pitch + (lane >> 4) * 16;
#pragma unroll
        for (int v = 0; v < VB; ++v) {
            const uint32_t block = warp + 4 * v;
            if (block >= blocks) break;
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                uint32_t b[4];
                ldmatrix4_trans(b, va + n * 16 * pitch + block * 32);
                mma_bf16(o[2 * v], pw[n], b[0], b[1]);
                mma_bf16(o[2 * v + 1], pw[n], b[2], b[3]);
            }
        }
        __syncthreads();
    }
    copy_wait<0>();
#pragma unroll
    for (int off = 1; off <= 2; off <<= 1) {
        l[0] += __shfl_xor_sync(0xFFFFFFFFu, l[0], off);
        l[1] += __shfl_xor_sync(0xFFFFFFFFu, l[1], off);
    }
    float* sums = tops + 4 * 16;
    if ((lane & 3) == 0) {
        sums[warp * 16 + (lane >> 2)] = l[0];
        sums[warp * 16 + (lane >> 2) + 8] = l[1];
    }
    __syncthreads();
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        const uint32_t row = (lane >> 2) + hf * 8;
        if (row >= nh) continue;
        if (warp == 0 && (lane & 3) == 0) {
            part_ml[(prow + row) * 2] = m[hf];
            part_ml[(prow + row) * 2 + 1] = (sums[row] + sums[16 + row]) + (sums[32 + row] + sums[48 + row]);
        }
        float* to = p.part + (prow + row) * p.rank4;
#pragma unroll
        for (int v = 0; v < VB; ++v) {
            const uint32_t block = warp + 4 * v;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const uint32_t col = block * 16 + half * 8 + (lane & 3) * 2;
                if (col < p.rank4)  // (rank4 is even; columns beyond the rank are not read)
                    *reinterpret_cast<float2*>(to + col) = make_float2(o[2 * v + half][hf * 2], o[2 * v + half][hf * 2 + 1]);
            }
        }
    }
}

// Smallest power of two of threads with four latent dimensions each.
__host__ __device__ inline uint32_t output_width(uint32_t kp) {
    uint32_t w = 16;
    while (w < kp / 4) w <<= 1;
    return w;
}

// CTA (head, block of value dimensions, row): the sum of latents, then its rows of W_uv_h.
template <typename TA>
__global__ void __launch_bounds__(128)
latent_output_kernel(const __grid_constant__ LatentParams p) {
    extern __shared__ __align__(16) float lat[];  // [groups][kp], zeros beyond the rank
    __shared__ float factor[kMaxSplits];
    pdl_launch_dependents();
    const LatentArgs& a = p.a;
    const LatentShape& s = a.s;
    const uint32_t h = blockIdx.x, v0 = blockIdx.y * kOutputRows, r = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t kp = a.up.kp, rows = min(kOutputRows, s.vdim - v0);
    const bf16* w = a.up.w + ((size_t)s.heads * s.dim + (size_t)h * s.vdim + v0) * kp;
    if (tid == 0) prefetch_l2_bulk(w, rows * kp * 2);
    pdl_wait();
    if (p.direct) {
        const TA* x = static_cast<const TA*>(p.direct) + (size_t)r * p.direct_pitch + (size_t)h * s.rank;
        for (uint32_t i = tid; i < kp; i += blockDim.x) lat[i] = i < s.rank ? from_act(x[i]) : 0.0f;
    } else {
        const uint32_t len = (uint32_t)a.pos[r] + 1;
        const uint32_t per = ((len + p.splits - 1) / p.splits + kTile - 1) / kTile * kTile, n = (len + per - 1) / per;
        const size_t row0 = (size_t)r * p.splits * s.heads + h;
        const float* ml = p.part + (size_t)p.rows * p.splits * s.heads * p.rank4;
        // every warp: lane i looks after ranges i and i + 32
        static_assert(kMaxSplits == 64, "two ranges per lane");
        float2 x = make_float2(-INFINITY, 0.0f), y = x;
        if (lane < n) x = *reinterpret_cast<const float2*>(ml + (row0 + (size_t)lane * s.heads) * 2);
        if (lane + 32 < n) y = *reinterpret_cast<const float2*>(ml + (row0 + (size_t)(lane + 32) * s.heads) * 2);
        float top = fmaxf(x.x, y.x);
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) top = fmaxf(top, __shfl_xor_sync(0xFFFFFFFFu, top, off));
        const float fx = exp2f(x.x - top), fy = exp2f(y.x - top), inv = 1.0f / warp_sum_f(fx * x.y + fy * y.y);
        if (warp == 0) {
            factor[lane] = fx * inv;
            factor[lane + 32] = fy * inv;
        }
        __syncthreads();
        // four dimensions per thread; short latents: groups of threads share the ranges
        const uint32_t width = min(128u, output_width(kp)), groups = 128 / width, g = tid / width;
        for (uint32_t c = tid % width; c < kp / 4; c += width) {
            float4 acc = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (4 * c < s.rank) {
                const float* x = p.part + row0 * p.rank4 + 4 * c;
                constexpr uint32_t AHEAD = 8;  // ranges requested together; the factors of those behind the last are 0
                for (uint32_t q0 = g; q0 < n; q0 += AHEAD * groups) {
                    float4 v[AHEAD];
#pragma unroll
                    for (uint32_t j = 0; j < AHEAD; ++j)
                        v[j] = *reinterpret_cast<const float4*>(x + (size_t)min(q0 + j * groups, n - 1) * s.heads * p.rank4);
#pragma unroll
                    for (uint32_t j = 0; j < AHEAD; ++j) {
                        const uint32_t q = q0 + j * groups;
                        const float f = q < n ? factor[q] : 0.0f;
                        acc.x = fmaf(f, v[j].x, acc.x);
                        acc.y = fmaf(f, v[j].y, acc.y);
                        acc.z = fmaf(f, v[j].z, acc.z);
                        acc.w = fmaf(f, v[j].w, acc.w);
                    }
                }
                if (4 * c + 1 >= s.rank) acc.y = 0.0f;
                if (4 * c + 2 >= s.rank) acc.z = 0.0f;
                if (4 * c + 3 >= s.rank) acc.w = 0.0f;
            }
            *reinterpret_cast<float4*>(lat + g * kp + 4 * c) = acc;
        }
        if (groups > 1) {
            __syncthreads();
            for (uint32_t i = tid; i < kp; i += 128) {
                float t = lat[i];
                for (uint32_t q = 1; q < groups; ++q) t += lat[q * kp + i];
                lat[i] = t;
            }
        }
    }
    __syncthreads();
    TA* out = static_cast<TA*>(a.out) + (size_t)r * a.out_pitch;
    constexpr uint32_t PER = kOutputRows / 4;  // value dimensions of a warp
    float acc[PER];
#pragma unroll
    for (uint32_t j = 0; j < PER; ++j) acc[j] = 0.0f;
    for (uint32_t c = lane; c < kp / 8; c += 32) {
        const float4 x = reinterpret_cast<const float4*>(lat + 8 * c)[0], y = reinterpret_cast<const float4*>(lat + 8 * c)[1];
        uint4 u[PER];
#pragma unroll
        for (uint32_t j = 0; j < PER; ++j) u[j] = __ldg(reinterpret_cast<const uint4*>(w + (size_t)min(warp + 4 * j, rows - 1) * kp) + c);
#pragma unroll
        for (uint32_t j = 0; j < PER; ++j) {
            float f[8];
            unpack8(u[j], f);
            acc[j] += (f[0] * x.x + f[1] * x.y) + (f[2] * x.z + f[3] * x.w) + ((f[4] * y.x + f[5] * y.y) + (f[6] * y.z + f[7] * y.w));
        }
    }
#pragma unroll
    for (uint32_t j = 0; j < PER; ++j) {
        const float t = warp_sum_f(acc[j]);
        const uint32_t v = warp + 4 * j;
        if (lane == 0 && v < rows) out[h * s.vdim + v0 + v] = to_act<TA>(t);
    }
    if (h == 0 && blockIdx.y == 0)
        for (uint32_t i = s.heads * s.vdim + tid; i < a.out_pitch; i += blockDim.x) out[i] = to_act<TA>(0.0f);
}

int done(cudaError_t e) { return e == cudaSuccess ? ZQ_OK : cuda_fail(e); }

constexpr uint32_t kSmemLimit = 220 * 1024;
uint32_t rank4_of(const LatentShape& s) { return pad_to(s.rank, 4); }
// Whether a tile of the decode kernel fits, and the latent into the warps' registers.
bool tiled(const LatentShape& s) { return s.rank <= 1024 && decode_smem(s.keyp, 1) <= kSmemLimit; }
uint32_t key_pitch(const LatentShape& s) { return pad_to(s.dim + s.rot, 16); }
uint32_t value_pitch(const LatentShape& s) { return pad_to(s.vdim, 16); }
uint32_t decode_splits(const LatentShape& s, uint32_t rows) {
    const uint32_t most = 2 * 148 / (rows * ((s.heads + 15) / 16)), n = (s.ctx + kTile - 1) / kTile;
    const uint32_t k = n < kMaxSplits ? n : kMaxSplits;
    return most < 1 ? 1 : k < most ? k : most;
}

// Areas of the work memory.
struct Areas {
    size_t q, part, keys, values, zero, total;
};
Areas areas(const LatentShape& s, uint32_t max_rows, bool f32) {
    auto up = [](size_t n) { return (n + 255) / 256 * 256; };
    Areas w{};
    const size_t per_row = s.keyp > key_pitch(s) ? s.keyp : key_pitch(s);
    w.part = up((size_t)max_rows * s.heads * per_row * act_bytes(f32));
    size_t part = 0;
    for (uint32_t r = 1; r <= max_rows; ++r) {  // rows * splits is largest somewhere in between
        const size_t n = (size_t)r * decode_splits(s, r) * s.heads * (rank4_of(s) + 2) * sizeof(float);
        if (n > part) part = n;
        if (decode_splits(s, r) == 1 && r >= kFoldRows) break;
    }
    const size_t many = (size_t)max_rows * s.heads * (rank4_of(s) + 2) * sizeof(float);  // one range per row
    const size_t direct = (size_t)max_rows * pad64(s.heads * s.rank) * act_bytes(f32);
    part = part > many ? part : many;
    part = part > direct ? part : direct;
    w.keys = w.part + up(part);
    w.values = w.keys + (f32 ? 0 : up((size_t)pad_to(s.ctx, kTile) * s.heads * key_pitch(s) * sizeof(bf16)));
    w.zero = w.values + (f32 ? 0 : up((size_t)pad_to(s.ctx, kTile) * s.heads * value_pitch(s) * sizeof(bf16)));
    w.total = w.zero + 256;
    return w;
}

template <typename TA>
int output(const LatentParams& p, cudaStream_t st) {
    const LatentShape& s = p.a.s;
    const dim3 grid(s.heads, (s.vdim + kOutputRows - 1) / kOutputRows, p.rows);
    const uint32_t w = output_width(p.a.up.kp), groups = w < 128 ? 128 / w : 1;
    return done(launch_pdl(latent_output_kernel<TA>, grid, dim3(128), groups * p.a.up.kp * sizeof(float), st, p));
}
template <typename TA>
int query(const LatentParams& p, cudaStream_t st) {
    const LatentShape& s = p.a.s;
    const dim3 grid(s.heads * p.rank_blocks + (p.a.own ? 1 : 0), p.rows);
    return done(launch_pdl(latent_query_kernel<TA>, grid, dim3(128), s.dim * sizeof(float), st, p));
}

template <int VB>
int decode(const LatentParams& p, cudaStream_t st) {
    const LatentShape& s = p.a.s;
    const uint32_t stages = decode_smem(s.keyp, 2) <= kSmemLimit ? 2 : 1, smem = decode_smem(s.keyp, stages);
    ZQ_CUDA(cudaFuncSetAttribute(latent_decode_kernel<VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemLimit));
    return done(launch_pdl(latent_decode_kernel<VB>, dim3(p.splits, (s.heads + 15) / 16, p.rows), dim3(128), smem, st, p, stages));
}

}  // namespace

size_t latent_work_bytes(const LatentShape& s, uint32_t max_rows, bool f32) { return areas(s, max_rows, f32).total; }

int launch_latent(const LatentArgs& a, uint32_t rows, bool one_sequence, uint32_t pos0, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    const LatentShape& s = a.s;
    if (s.rank > 1024 || s.dim > 4096 || s.rot > kMaxRot) return ZQ_ERR_LIMIT;
    if (rows > a.max_rows || rows > 65535) return ZQ_ERR_BAD_ARG;
    const Areas w = areas(s, a.max_rows, f32);
    char* work = static_cast<char*>(a.work);
    LatentParams p{};
    p.a = a;
    p.scale2 = a.scale * kLog2e;
    p.rows = rows;
    p.rank_blocks = (s.rank + kQueryRanks - 1) / kQueryRanks;
    p.q = work;
    p.part = reinterpret_cast<float*>(work + w.part);
    p.rank4 = rank4_of(s);
    int rc;
    const bool expand = !f32 && one_sequence && rows > kFoldRows && key_pitch(s) <= 256 && value_pitch(s) <= 256;
    if (expand) {
        p.q_pitch = key_pitch(s);
        p.v_pitch = value_pitch(s);
        p.keys = reinterpret_cast<bf16*>(work + w.keys);
        p.values = reinterpret_cast<bf16*>(work + w.values);
        p.zero = reinterpret_cast<int32_t*>(work + w.zero);
        p.tokens = pos0 + rows;
        const dim3 grid(rows, a.own ? 2 : 1);
        const bool pairs = s.dim % 2 == 0 && a.ld % 2 == 0;
        rc = done(pairs ? launch_pdl(latent_rows_kernel<true>, grid, dim3(256), 0, st, p)
                        : launch_pdl(latent_rows_kernel<false>, grid, dim3(256), 0, st, p));
        if (rc != ZQ_OK) return rc;
        const HeadSplit split{p.keys, p.values, s.heads, s.dim, s.vdim, p.q_pitch, p.v_pitch};
        const bf16* rows_of_slot = static_cast<const bf16*>(a.cache) + (size_t)a.slot0 * s.ctx * s.keyp;
        if ((rc = launch_gemm_bf16_heads(a.up, rows_of_slot, s.keyp, p.tokens, p.tokens, split, st)) != ZQ_OK) return rc;
        if ((rc = done(launch_pdl(latent_key_part_kernel, dim3(pad_to(p.tokens, kTile)), dim3(128), 0, st, p))) != ZQ_OK) return rc;
        const GqaShape g{s.heads, s.heads, s.dim + s.rot, s.vdim, p.q_pitch, p.v_pitch, pad_to(s.ctx, kTile), 1};
        return launch_gqa_attention(g, p.q, p.keys, p.values, a.out, a.out_pitch, a.scale, a.pos, p.zero, rows, true, pos0, nullptr,
                                    false, st);
    }
    p.q_pitch = s.keyp;
    if ((rc = f32 ? query<float>(p, st) : query<bf16>(p, st)) != ZQ_OK) return rc;
    if (f32 || !tiled(s)) {
        GqaShape g{s.heads, 1, s.rank + s.rot, s.rank, s.keyp, s.keyp, s.ctx, s.slots};  // the values are the key rows' front
        p.direct = p.part;
        p.direct_pitch = pad64(s.heads * s.rank);
        if ((rc = launch_gqa_plain(g, p.q, a.cache, a.cache, p.part, p.direct_pitch, a.scale, a.pos, a.slots, rows, f32, st)) != ZQ_OK)
            return rc;
        return f32 ? output<float>(p, st) : output<bf16>(p, st);
    }
    p.splits = decode_splits(s, rows);
    const uint32_t blocks = ((s.rank + 15) / 16 + 3) / 4;
    rc = blocks <= 2 ? decode<2>(p, st) : blocks <= 4 ? decode<4>(p, st) : blocks <= 8 ? decode<8>(p, st) : decode<16>(p, st);
    return rc != ZQ_OK ? rc : output<bf16>(p, st);
}

}  // namespace zq
