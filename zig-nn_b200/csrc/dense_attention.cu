// Causal grouped-query attention over a per-slot key / value cache, softmax in f32.
//   * prefill (bf16), many rows: tcgen05, dense_attention_tc.cu;
//   * prefill (bf16), few rows: tiles of 64 packed query rows (token, head of the group) against tiles of 64 keys, mma.sync on
//     bf16 operands with f32 accumulation, keys and values double-buffered by cp.async;
//   * decode (bf16): a CTA per (row, key head, key range): the group's heads are the 16 rows of the MMAs, the four
//     warps share each tile of 64 keys; the ranges meet in a second small kernel. The query and key norms, the value
//     mixing and the cache write of the new token happen in the same kernel;
//   * f32, and heads beyond 256 dimensions: one warp-parallel online softmax per (row, head), plain multiply-adds.
// A weight is rounded to bf16 for its product with the values; the sum it is divided by adds the same rounded weights.
#include "dense.h"
#include "tile_common.cuh"

namespace zq {
namespace {

constexpr uint32_t kTile = 64;  // keys per tile

// Keys (or values) [k0, k0 + kTile) of one head -> shared memory rows of pitch (dp + 8) halves; zeros beyond k_end.
__device__ __forceinline__ void load_tile(uint32_t dst, const bf16* cache, uint32_t kv_heads, uint32_t g, uint32_t dp,
                                          uint32_t k0, uint32_t k_end) {
    const uint32_t cpr = dp / 8, pitch = (dp + 8) * 2;
    const uint32_t dr = blockDim.x / cpr, dc = blockDim.x % cpr;
    uint32_t row = threadIdx.x / cpr, c = threadIdx.x % cpr;
    while (row < kTile) {
        const uint32_t key = k0 + row;
        const bool ok = key < k_end;
        copy16(dst + row * pitch + c * 16, cache + ((size_t)(ok ? key : k0) * kv_heads + g) * dp + c * 8, ok);
        row += dr;
        c += dc;
        if (c >= cpr) {
            c -= cpr;
            ++row;
        }
    }
}

// Query fragments of 16 packed rows. row_ptr(i): row i of the 16 (null: zeros).
template <int KS, typename RowPtr>
__device__ __forceinline__ void load_q(uint32_t (&q)[KS][4], uint32_t ks, RowPtr row_ptr) {
    const uint32_t lane = threadIdx.x & 31;
    const bf16 *r0 = row_ptr(lane >> 2), *r1 = row_ptr((lane >> 2) + 8);
#pragma unroll
    for (int kk = 0; kk < KS; ++kk) {
        const uint32_t col = kk * 16 + (lane & 3) * 2;
        const bool in = (uint32_t)kk < ks;
        q[kk][0] = in && r0 ? *reinterpret_cast<const uint32_t*>(r0 + col) : 0u;
        q[kk][1] = in && r1 ? *reinterpret_cast<const uint32_t*>(r1 + col) : 0u;
        q[kk][2] = in && r0 ? *reinterpret_cast<const uint32_t*>(r0 + col + 8) : 0u;
        q[kk][3] = in && r1 ? *reinterpret_cast<const uint32_t*>(r1 + col + 8) : 0u;
    }
}

// One step of the online softmax of a warp's 16 rows over NK * 16 keys starting `key_row` rows into the tile.
// Lane holds rows lane / 4 and lane / 4 + 8; lim0 / lim1: keys of the tile that these rows may see (counted from key_row).
template <int KS, int VS, int NK>
__device__ __forceinline__ void attend(const uint32_t (&q)[KS][4], float (&o)[VS * 2][4], float (&m)[2], float (&l)[2],
                                       uint32_t k_tile, uint32_t v_tile, uint32_t key_row, uint32_t dimp, uint32_t vdimp,
                                       float scale2, int lim0, int lim1, bool masked) {
    const uint32_t lane = threadIdx.x & 31;
    const uint32_t kpitch = (dimp + 8) * 2, vpitch = (vdimp + 8) * 2;
    float s[NK * 2][4];
#pragma unroll
    for (int n = 0; n < NK * 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[n][e] = 0.0f;
    const uint32_t kaddr = k_tile + (key_row + ((lane >> 4) << 3) + (lane & 7)) * kpitch + ((lane >> 3) & 1) * 16;
#pragma unroll
    for (int kk = 0; kk < KS; ++kk) {
        if (kk * 16u >= dimp) break;
#pragma unroll
        for (int n = 0; n < NK; ++n) {
            uint32_t b[4];
            ldmatrix4(b, kaddr + n * 16 * kpitch + kk * 32);
            mma_bf16(s[2 * n], q[kk], b[0], b[1]);
            mma_bf16(s[2 * n + 1], q[kk], b[2], b[3]);
        }
    }
    float mx0 = m[0], mx1 = m[1];
#pragma unroll
    for (int n = 0; n < NK * 2; ++n) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            s[n][e] *= scale2;
            if (masked) {
                const int col = n * 8 + (lane & 3) * 2 + (e & 1);
                if (col >= (e < 2 ? lim0 : lim1)) s[n][e] = -INFINITY;
            }
        }
        mx0 = fmaxf(mx0, fmaxf(s[n][0], s[n][1]));
        mx1 = fmaxf(mx1, fmaxf(s[n][2], s[n][3]));
    }
#pragma unroll
    for (int off = 1; off <= 2; off <<= 1) {
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xFFFFFFFFu, mx0, off));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xFFFFFFFFu, mx1, off));
    }
    const float b0 = mx0 == -INFINITY ? 0.0f : mx0, b1 = mx1 == -INFINITY ? 0.0f : mx1;
    const float f0 = exp2f(m[0] - b0), f1 = exp2f(m[1] - b1);
    m[0] = mx0;
    m[1] = mx1;
    float a0 = 0.0f, a1 = 0.0f;
    uint32_t p[NK][4];
#pragma unroll
    for (int n = 0; n < NK; ++n) {
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            const float* t = s[2 * n + hf];
            const uint32_t top = pack_bf16(exp2f(t[0] - b0), exp2f(t[1] - b0)), bot = pack_bf16(exp2f(t[2] - b1), exp2f(t[3] - b1));
            a0 += bf16_lo(top) + bf16_hi(top);
            a1 += bf16_lo(bot) + bf16_hi(bot);
            p[n][2 * hf] = top;
            p[n][2 * hf + 1] = bot;
        }
    }
    l[0] = l[0] * f0 + a0;  // this lane's share of the sums; the four lanes of a row meet at the end
    l[1] = l[1] * f1 + a1;
#pragma unroll
    for (int v = 0; v < VS * 2; ++v) {
        o[v][0] *= f0; o[v][1] *= f0; o[v][2] *= f1; o[v][3] *= f1;
    }
    const uint32_t vaddr = v_tile + (key_row + ((lane >> 3) & 1) * 8 + (lane & 7)) * vpitch + (lane >> 4) * 16;
#pragma unroll
    for (int v = 0; v < VS; ++v) {
        if (v * 16u >= vdimp) break;
#pragma unroll
        for (int n = 0; n < NK; ++n) {
            uint32_t b[4];
            ldmatrix4_trans(b, vaddr + n * 16 * vpitch + v * 32);
            mma_bf16(o[2 * v], p[n], b[0], b[1]);
            mma_bf16(o[2 * v + 1], p[n], b[2], b[3]);
        }
    }
}

struct AttnArgs {
    GqaShape s;
    const bf16 *q, *kc, *vc;
    bf16* out;
    uint32_t out_pitch;
    float scale2;  // scale * log2(e)
    const int32_t *pos, *slots;
    uint32_t rows, pos0, splits;
    float* part;  // decode: [rows][splits][heads][vdimp] values, then [rows][splits][heads][2] maximum and sum
    // decode with the steps ahead of it (null qkv: q and the row's own key and value are there already)
    QkvPostArgs pre;
};

__device__ __forceinline__ void zero_pad(bf16* out_row, uint32_t from, uint32_t pitch) {
    for (uint32_t i = from + threadIdx.x; i < pitch; i += blockDim.x) out_row[i] = __float2bfloat16_rn(0.0f);
}

template <int D>
__global__ void __launch_bounds__(128)
gqa_prefill_kernel(const __grid_constant__ AttnArgs a) {
    constexpr int S = D / 16;
    extern __shared__ __align__(16) unsigned char sm[];
    pdl_launch_dependents();
    pdl_wait();
    const GqaShape& s = a.s;
    const uint32_t R = s.heads / s.kv_heads, g = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t n_rows = a.rows * R;  // packed rows of this key head
    const uint32_t m0 = (gridDim.x - 1 - blockIdx.x) * 64;  // the longest tiles first
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(sm);
    const uint32_t kbytes = kTile * (s.dimp + 8) * 2, vbytes = kTile * (s.vdimp + 8) * 2;
    auto ktile = [&](uint32_t b) { return base + b * (kbytes + vbytes); };
    auto vtile = [&](uint32_t b) { return base + b * (kbytes + vbytes) + kbytes; };
    const size_t slot = (size_t)(uint32_t)a.slots[0] * s.ctx;
    const bf16* kc = a.kc + slot * s.kv_heads * s.dimp;
    const bf16* vc = a.vc + slot * s.kv_heads * s.vdimp;

    const uint32_t last = min(m0 + 64, n_rows) - 1;
    const uint32_t k_end = a.pos0 + last / R + 1;
    const uint32_t n_tiles = (k_end + kTile - 1) / kTile;
    load_tile(ktile(0), kc, s.kv_heads, g, s.dimp, 0, k_end);
    load_tile(vtile(0), vc, s.kv_heads, g, s.vdimp, 0, k_end);
    copy_commit();

    const uint32_t w0 = m0 + warp * 16;
    uint32_t q[S][4];
    load_q<S>(q, s.dimp / 16, [&](uint32_t i) -> const bf16* {
        const uint32_t mrow = w0 + i;
        return mrow < n_rows ? a.q + ((size_t)(mrow / R) * s.heads + g * R + mrow % R) * s.dimp : nullptr;
    });
    float o[S * 2][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int v = 0; v < S * 2; ++v)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[v][e] = 0.0f;
    const uint32_t r0 = w0 + (lane >> 2), r1 = r0 + 8;
    const uint32_t see0 = r0 < n_rows ? a.pos0 + r0 / R + 1 : 0, see1 = r1 < n_rows ? a.pos0 + r1 / R + 1 : 0;
    const uint32_t see_all = a.pos0 + w0 / R + 1;  // keys that every row of the warp sees
    for (uint32_t t = 0; t < n_tiles; ++t) {
        if (t + 1 < n_tiles) {
            load_tile(ktile((t + 1) & 1), kc, s.kv_heads, g, s.dimp, (t + 1) * kTile, k_end);
            load_tile(vtile((t + 1) & 1), vc, s.kv_heads, g, s.vdimp, (t + 1) * kTile, k_end);
        }
        copy_commit();
        copy_wait<1>();
        __syncthreads();
        const uint32_t k0 = t * kTile;
        if (w0 < n_rows)
            attend<S, S, 4>(q, o, m, l, ktile(t & 1), vtile(t & 1), 0, s.dimp, s.vdimp, a.scale2, (int)see0 - (int)k0,
                            (int)see1 - (int)k0, k0 + kTile > see_all || w0 + 16 > n_rows);
        __syncthreads();
    }
#pragma unroll
    for (int off = 1; off <= 2; off <<= 1) {
        l[0] += __shfl_xor_sync(0xFFFFFFFFu, l[0], off);
        l[1] += __shfl_xor_sync(0xFFFFFFFFu, l[1], off);
    }
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        const uint32_t row = hf ? r1 : r0;
        if (row >= n_rows) continue;
        const uint32_t head = g * R + row % R;
        bf16* out = a.out + (size_t)(row / R) * a.out_pitch + (size_t)head * s.vdim;
        const float inv = 1.0f / l[hf];
#pragma unroll
        for (int v = 0; v < S * 2; ++v) {
            const uint32_t col = v * 8 + (lane & 3) * 2;
            if (col < s.vdim) out[col] = __float2bfloat16_rn(o[v][hf * 2] * inv);
            if (col + 1 < s.vdim) out[col + 1] = __float2bfloat16_rn(o[v][hf * 2 + 1] * inv);
        }
    }
    if (g == 0)  // columns beyond the heads
        for (uint32_t t = m0 / R; t <= last / R; ++t) zero_pad(a.out + (size_t)t * a.out_pitch, s.heads * s.vdim, a.out_pitch);
}

constexpr uint32_t kDecodeStages = 3;

template <int D>
__global__ void __launch_bounds__(128)
gqa_decode_kernel(const __grid_constant__ AttnArgs a) {
    constexpr int S = D / 16;
    extern __shared__ __align__(16) unsigned char sm[];
    pdl_launch_dependents();
    pdl_wait();
    const GqaShape& s = a.s;
    const uint32_t R = s.heads / s.kv_heads, m_tiles = (R + 15) / 16;
    const uint32_t split = blockIdx.x, g = blockIdx.y / m_tiles, h0 = (blockIdx.y % m_tiles) * 16, r = blockIdx.z;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t len = (uint32_t)a.pos[r] + 1;
    const uint32_t per = ((len + a.splits - 1) / a.splits + kTile - 1) / kTile * kTile;
    const uint32_t k_begin = split * per, k_end = min(len, k_begin + per);
    const uint32_t nh = min(16u, R - h0);  // heads of this CTA
    float* part_ml = a.part + (size_t)a.rows * a.splits * s.heads * s.vdimp;
    const size_t prow = ((size_t)r * a.splits + split) * s.heads + g * R + h0;
    if (k_begin >= k_end) {
        for (uint32_t i = threadIdx.x; i < nh; i += blockDim.x) {
            part_ml[(prow + i) * 2] = -INFINITY;
            part_ml[(prow + i) * 2 + 1] = 0.0f;
        }
        return;
    }
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(sm);
    const uint32_t kbytes = kTile * (s.dimp + 8) * 2, vbytes = kTile * (s.vdimp + 8) * 2;
    auto ktile = [&](uint32_t b) { return base + (b % kDecodeStages) * (kbytes + vbytes); };
    auto vtile = [&](uint32_t b) { return ktile(b) + kbytes; };
    const size_t slot = (size_t)(uint32_t)a.slots[r] * s.ctx;
    const bf16* kc = a.kc + slot * s.kv_heads * s.dimp;
    const bf16* vc = a.vc + slot * s.kv_heads * s.vdimp;
    const uint32_t n_tiles = (k_end - k_begin + kTile - 1) / kTile;
    // With `pre`, the row's own key and value are made here, by the CTA whose range ends with them: its copies stop
    // ahead of them.
    const bool fused = a.pre.qkv != nullptr, own = fused && k_end == len;
    const uint32_t c_end = own ? k_end - 1 : k_end;
#pragma unroll
    for (uint32_t t = 0; t + 1 < kDecodeStages; ++t) {
        if (t < n_tiles) {
            load_tile(ktile(t), kc, s.kv_heads, g, s.dimp, k_begin + t * kTile, c_end);
            load_tile(vtile(t), vc, s.kv_heads, g, s.vdimp, k_begin + t * kTile, c_end);
        }
        copy_commit();
    }
    bf16* own_q = reinterpret_cast<bf16*>(sm + kDecodeStages * (kbytes + vbytes));  // [16][dimp], then own key and value
    bf16 *own_k = own_q + 16 * s.dimp, *own_v = own_k + s.dimp;
    if (fused) {
        const QkvPostArgs& f = a.pre;
        const float* row = f.qkv + (size_t)r * ((s.heads + s.kv_heads) * s.dim + s.kv_heads * s.vdim);
        const float temp = query_temperature(len - 1, f.temp_coef, f.temp_every);
        for (uint32_t i = warp; i < nh + (own ? 2 : 0); i += 4) {
            if (i < nh) {
                norm_head(row + (size_t)(g * R + h0 + i) * s.dim, f.q_norm, s.dim, s.dimp, f.eps, temp, own_q + i * s.dimp, lane);
            } else if (i == nh) {
                norm_head(row + (size_t)(s.heads + g) * s.dim, f.k_norm, s.dim, s.dimp, f.eps, 1.0f, own_k, lane);
                __syncwarp();
                bf16* o = const_cast<bf16*>(kc) + ((size_t)(len - 1) * s.kv_heads + g) * s.dimp;
                for (uint32_t e = lane; e < s.dimp; e += 32) o[e] = own_k[e];
            } else {
                const float* v = row + (size_t)(s.heads + s.kv_heads) * s.dim + (size_t)g * s.vdim;
                float* first = f.v_first ? f.v_first + ((size_t)r * s.kv_heads + g) * s.vdim : nullptr;
                bf16* o = const_cast<bf16*>(vc) + ((size_t)(len - 1) * s.kv_heads + g) * s.vdimp;
                for (uint32_t e = lane; e < s.vdimp; e += 32)
                    own_v[e] = o[e] = to_act<bf16>(e < s.vdim ? mixed_value(v[e], f.vmix, first, e) : 0.0f);
            }
        }
        __syncthreads();
    }
    uint32_t q[S][4];
    load_q<S>(q, s.dimp / 16, [&](uint32_t i) -> const bf16* {
        if (i >= nh) return nullptr;
        return fused ? own_q + i * s.dimp : a.q + ((size_t)r * s.heads + g * R + h0 + i) * s.dimp;
    });
    float o[S * 2][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int v = 0; v < S * 2; ++v)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[v][e] = 0.0f;
    for (uint32_t t = 0; t < n_tiles; ++t) {
        const uint32_t ahead = t + kDecodeStages - 1;
        if (ahead < n_tiles) {
            load_tile(ktile(ahead), kc, s.kv_heads, g, s.dimp, k_begin + ahead * kTile, c_end);
            load_tile(vtile(ahead), vc, s.kv_heads, g, s.vdimp, k_begin + ahead * kTile, c_end);
        }
        copy_commit();
        copy_wait<kDecodeStages - 1>();
        __syncthreads();
        if (own && t + 1 == n_tiles) {  // the place behind the copied keys
            const uint32_t at = k_end - 1 - (k_begin + t * kTile);
            unsigned char* kt = sm + (t % kDecodeStages) * (kbytes + vbytes) + at * (s.dimp + 8) * 2;
            unsigned char* vt = sm + (t % kDecodeStages) * (kbytes + vbytes) + kbytes + at * (s.vdimp + 8) * 2;
            for (uint32_t e = threadIdx.x; e < s.dimp; e += blockDim.x) reinterpret_cast<bf16*>(kt)[e] = own_k[e];
            for (uint32_t e = threadIdx.x; e < s.vdimp; e += blockDim.x) reinterpret_cast<bf16*>(vt)[e] = own_v[e];
            __syncthreads();
        }
        const int lim = (int)(k_end - k_begin) - (int)(t * kTile + warp * 16);
        attend<S, S, 1>(q, o, m, l, ktile(t), vtile(t), warp * 16, s.dimp, s.vdimp, a.scale2, lim, lim, lim < 16);
        __syncthreads();
    }
#pragma unroll
    for (int off = 1; off <= 2; off <<= 1) {
        l[0] += __shfl_xor_sync(0xFFFFFFFFu, l[0], off);
        l[1] += __shfl_xor_sync(0xFFFFFFFFu, l[1], off);
    }
    // the four warps' shares meet in shared memory (the tiles are no longer needed)
    copy_wait<0>();
    __syncthreads();
    float* ml = reinterpret_cast<float*>(sm);          // [4 warps][16 rows][2]
    float* ov = ml + 4 * 16 * 2;                       // [4 warps][16 rows][vdimp]
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        const uint32_t row = (lane >> 2) + hf * 8;
        if ((lane & 3) == 0) {
            ml[(warp * 16 + row) * 2] = m[hf];
            ml[(warp * 16 + row) * 2 + 1] = l[hf];
        }
#pragma unroll
        for (int v = 0; v < S * 2; ++v) {
            const uint32_t col = v * 8 + (lane & 3) * 2;
            if (col < s.vdimp)
                *reinterpret_cast<float2*>(ov + (size_t)(warp * 16 + row) * s.vdimp + col) =
                    make_float2(o[v][hf * 2], o[v][hf * 2 + 1]);
        }
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < nh * s.vdimp; i += blockDim.x) {
        const uint32_t row = i / s.vdimp, col = i % s.vdimp;
        float mx = -INFINITY;
#pragma unroll
        for (uint32_t w = 0; w < 4; ++w) mx = fmaxf(mx, ml[(w * 16 + row) * 2]);
        float sum = 0.0f, acc = 0.0f;
#pragma unroll
        for (uint32_t w = 0; w < 4; ++w) {
            const float f = exp2f(ml[(w * 16 + row) * 2] - mx);
            sum += f * ml[(w * 16 + row) * 2 + 1];
            acc += f * ov[(size_t)(w * 16 + row) * s.vdimp + col];
        }
        if (a.splits == 1) {
            if (col < s.vdim)
                a.out[(size_t)r * a.out_pitch + (size_t)(g * R + h0 + row) * s.vdim + col] = __float2bfloat16_rn(acc / sum);
        } else {
            a.part[(prow + row) * s.vdimp + col] = acc;
            if (col == 0) {
                part_ml[(prow + row) * 2] = mx;
                part_ml[(prow + row) * 2 + 1] = sum;
            }
        }
    }
    if (a.splits == 1 && blockIdx.y == 0) zero_pad(a.out + (size_t)r * a.out_pitch, s.heads * s.vdim, a.out_pitch);
}

__device__ __forceinline__ uint32_t pad32(uint32_t n) { return (n + 31u) & ~31u; }

// The key ranges of a row and head: out = sum of their values, each brought to the common maximum, over their sums.
__global__ void __launch_bounds__(256)
gqa_combine_kernel(const __grid_constant__ AttnArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const GqaShape& s = a.s;
    const uint32_t h = blockIdx.x, r = blockIdx.y, lane = threadIdx.x & 31;
    const float* part_ml = a.part + (size_t)a.rows * a.splits * s.heads * s.vdimp;
    // the ranges that hold keys come first; lane i keeps the factor of range i (at most 32 of them)
    const uint32_t len = (uint32_t)a.pos[r] + 1;
    const uint32_t per = ((len + a.splits - 1) / a.splits + kTile - 1) / kTile * kTile, n = (len + per - 1) / per;
    const size_t row0 = (size_t)r * a.splits * s.heads + h;
    const float2 ml = lane < n ? *reinterpret_cast<const float2*>(part_ml + (row0 + (size_t)lane * s.heads) * 2) : make_float2(-INFINITY, 0.0f);
    float mx = ml.x;
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, off));
    const float f = exp2f(ml.x - mx), inv = 1.0f / warp_sum_f(f * ml.y);
    bf16* out = a.out + (size_t)r * a.out_pitch;
    for (uint32_t d = threadIdx.x; d < pad32(s.vdim); d += blockDim.x) {
        float acc = 0.0f;
#pragma unroll 8
        for (uint32_t i = 0; i < n; ++i) {
            const float v = d < s.vdim ? a.part[(row0 + (size_t)i * s.heads) * s.vdimp + d] : 0.0f;
            acc = fmaf(__shfl_sync(0xFFFFFFFFu, f, i), v, acc);
        }
        if (d < s.vdim) out[(size_t)h * s.vdim + d] = __float2bfloat16_rn(acc * inv);
    }
    if (h == 0) zero_pad(out, s.heads * s.vdim, a.out_pitch);
}

// One (row, head) per CTA: the four warps take tiles of 32 keys in turn, a key per lane for the scores, VR value
// dimensions per lane for the accumulation.
template <typename TA, int VR>
__global__ void __launch_bounds__(128)
gqa_plain_kernel(GqaShape s, const TA* __restrict__ q, const TA* __restrict__ kc, const TA* __restrict__ vc, TA* __restrict__ out,
                 uint32_t out_pitch, float scale, const int32_t* __restrict__ pos, const int32_t* __restrict__ slots) {
    extern __shared__ __align__(16) float smf[];
    pdl_launch_dependents();
    pdl_wait();
    float* qs = smf;                   // [dimp]
    float* ml = qs + s.dimp;           // [4][2]
    float* ov = ml + 8;                // [4][32 * VR]
    const uint32_t r = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const uint32_t g = h / (s.heads / s.kv_heads), len = (uint32_t)pos[r] + 1;
    const size_t slot = (size_t)(uint32_t)slots[r] * s.ctx;
    for (uint32_t i = threadIdx.x; i < s.dimp; i += blockDim.x) qs[i] = from_act(q[((size_t)r * s.heads + h) * s.dimp + i]);
    __syncthreads();
    float m = -INFINITY, l = 0.0f, o[VR];
#pragma unroll
    for (int v = 0; v < VR; ++v) o[v] = 0.0f;
    for (uint32_t k0 = warp * 32; k0 < len; k0 += 128) {
        const uint32_t key = k0 + lane;
        float sc = -INFINITY;
        if (key < len) {
            const TA* kr = kc + ((slot + key) * s.kv_heads + g) * s.dimp;
            float acc = 0.0f;
            for (uint32_t i = 0; i < s.dimp; i += 8) {
                float f[8];
                load8(kr + i, f);
#pragma unroll
                for (int e = 0; e < 8; ++e) acc = fmaf(qs[i + e], f[e], acc);
            }
            sc = acc * scale;
        }
        float mx = sc;
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, off));
        mx = fmaxf(mx, m);
        const float f = expf(m - mx), p = key < len ? expf(sc - mx) : 0.0f;
        m = mx;
        l = l * f + warp_sum_f(p);
#pragma unroll
        for (int v = 0; v < VR; ++v) o[v] *= f;
        const uint32_t n = min(32u, len - k0);
        for (uint32_t j = 0; j < n; ++j) {
            const float pj = __shfl_sync(0xFFFFFFFFu, p, j);
            const TA* vr = vc + ((slot + k0 + j) * s.kv_heads + g) * s.vdimp;
#pragma unroll
            for (int v = 0; v < VR; ++v) {
                const uint32_t d = lane + v * 32;
                if (d < s.vdim) o[v] = fmaf(pj, from_act(vr[d]), o[v]);
            }
        }
    }
    if (lane == 0) {
        ml[warp * 2] = m;
        ml[warp * 2 + 1] = l;
    }
#pragma unroll
    for (int v = 0; v < VR; ++v) ov[warp * 32 * VR + v * 32 + lane] = o[v];
    __syncthreads();
    TA* row = out + (size_t)r * out_pitch;
    const float mx = fmaxf(fmaxf(ml[0], ml[2]), fmaxf(ml[4], ml[6]));
    for (uint32_t d = threadIdx.x; d < s.vdim; d += blockDim.x) {
        float sum = 0.0f, acc = 0.0f;
#pragma unroll
        for (uint32_t w = 0; w < 4; ++w) {
            const float f = ml[w * 2] == -INFINITY ? 0.0f : expf(ml[w * 2] - mx);
            sum += f * ml[w * 2 + 1];
            acc += f * ov[w * 32 * VR + d];
        }
        row[(size_t)h * s.vdim + d] = to_act<TA>(acc / sum);
    }
    if (h == 0)
        for (uint32_t i = s.heads * s.vdim + threadIdx.x; i < out_pitch; i += blockDim.x) row[i] = to_act<TA>(0.0f);
}

int done(cudaError_t e) { return e == cudaSuccess ? ZQ_OK : cuda_fail(e); }

template <typename TA>
int plain_rows(const GqaShape& s, const void* q, const void* kc, const void* vc, void* out, uint32_t out_pitch, float scale,
          const int32_t* pos, const int32_t* slots, uint32_t rows, cudaStream_t st) {
    const dim3 grid(rows, s.heads);
    auto go = [&](auto kern, uint32_t vr) {
        const size_t smem = (s.dimp + 8 + 4 * 32 * vr) * sizeof(float);
        return done(launch_pdl(kern, grid, dim3(128), smem, st, s, static_cast<const TA*>(q), static_cast<const TA*>(kc),
                               static_cast<const TA*>(vc), static_cast<TA*>(out), out_pitch, scale, pos, slots));
    };
    if (s.vdim <= 64) return go(gqa_plain_kernel<TA, 2>, 2);
    if (s.vdim <= 256) return go(gqa_plain_kernel<TA, 8>, 8);
    return go(gqa_plain_kernel<TA, 32>, 32);
}

uint32_t decode_splits(const GqaShape& s) {
    const uint32_t n = (s.ctx + 255) / 256;
    return n < 1 ? 1 : n > 32 ? 32 : n;
}

template <int D>
int tiles_launch(AttnArgs& a, bool one_sequence, cudaStream_t st) {
    const GqaShape& s = a.s;
    const uint32_t R = s.heads / s.kv_heads;
    const uint32_t tile = kTile * (s.dimp + 8 + s.vdimp + 8) * 2;
    if (one_sequence && a.rows > 1) {
        // more than one of the small kernel's tiles: the tensor cores (their copies want 128-byte cache rows)
        if (a.rows * R > 64 && s.kv_heads * s.dimp >= 64 && s.kv_heads * s.vdimp >= 64) {
            const int rc = launch_gqa_prefill_tc(s, a.q, a.kc, a.vc, a.out, a.out_pitch, a.scale2, a.slots, a.rows, a.pos0, st);
            if (rc != ZQ_ERR_UNSUPPORTED) return rc;
        }
        ZQ_CUDA(cudaFuncSetAttribute(gqa_prefill_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, 2 * tile));
        return done(launch_pdl(gqa_prefill_kernel<D>, dim3((a.rows * R + 63) / 64, s.kv_heads), dim3(128), 2 * tile, st, a));
    }
    uint32_t smem = kDecodeStages * tile + (17 * s.dimp + s.vdimp) * 2;
    const uint32_t meet = (4 * 16 * 2 + 4 * 16 * s.vdimp) * 4;
    if (smem < meet) smem = meet;
    a.splits = decode_splits(s);
    ZQ_CUDA(cudaFuncSetAttribute(gqa_decode_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    int rc = done(launch_pdl(gqa_decode_kernel<D>, dim3(a.splits, s.kv_heads * ((R + 15) / 16), a.rows), dim3(128), smem, st, a));
    if (rc != ZQ_OK || a.splits == 1) return rc;
    return done(launch_pdl(gqa_combine_kernel, dim3(s.heads, a.rows), dim3(s.vdim >= 256 ? 256 : pad_to(s.vdim, 32)), 0, st, a));
}

}  // namespace

size_t gqa_work_bytes(const GqaShape& s, uint32_t max_rows) {
    const size_t n = decode_splits(s);
    return (size_t)max_rows * n * s.heads * (s.vdimp + 2) * sizeof(float);
}

static bool tiled(const GqaShape& s) { return s.dimp <= 256 && s.vdimp <= 256; }

static int attention_tiles(AttnArgs& a, bool one_sequence, cudaStream_t st) {
    const uint32_t d = a.s.dimp > a.s.vdimp ? a.s.dimp : a.s.vdimp;
    if (d <= 64) return tiles_launch<64>(a, one_sequence, st);
    if (d <= 128) return tiles_launch<128>(a, one_sequence, st);
    return tiles_launch<256>(a, one_sequence, st);
}

int launch_gqa_layer(const QkvPostArgs& p, void* out, uint32_t out_pitch, float scale, uint32_t rows, bool one_sequence,
                     uint32_t pos0, void* work, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    const GqaShape& s = p.s;
    if (f32 || !tiled(s) || (one_sequence && rows > 1)) {
        const int rc = launch_qkv_post(p, rows, f32, st);
        return rc != ZQ_OK ? rc
                           : launch_gqa_attention(s, p.q, p.kc, p.vc, out, out_pitch, scale, p.pos, p.slots, rows, one_sequence,
                                                  pos0, work, f32, st);
    }
    AttnArgs a{};
    a.s = s;
    a.kc = static_cast<const bf16*>(p.kc);
    a.vc = static_cast<const bf16*>(p.vc);
    a.out = static_cast<bf16*>(out);
    a.out_pitch = out_pitch;
    a.scale2 = scale * kLog2e;
    a.pos = p.pos;
    a.slots = p.slots;
    a.rows = rows;
    a.part = static_cast<float*>(work);
    a.pre = p;
    return attention_tiles(a, one_sequence, st);
}

int launch_gqa_plain(const GqaShape& s, const void* q, const void* kc, const void* vc, void* out, uint32_t out_pitch, float scale,
                     const int32_t* pos, const int32_t* slots, uint32_t rows, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    if (s.vdim > 1024 || s.dim > 4096) return ZQ_ERR_LIMIT;
    return f32 ? plain_rows<float>(s, q, kc, vc, out, out_pitch, scale, pos, slots, rows, st)
               : plain_rows<bf16>(s, q, kc, vc, out, out_pitch, scale, pos, slots, rows, st);
}

int launch_gqa_attention(const GqaShape& s, const void* q, const void* kc, const void* vc, void* out, uint32_t out_pitch,
                         float scale, const int32_t* pos, const int32_t* slots, uint32_t rows, bool one_sequence,
                         uint32_t pos0, void* work, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    if (f32 || !tiled(s)) return launch_gqa_plain(s, q, kc, vc, out, out_pitch, scale, pos, slots, rows, f32, st);
    AttnArgs a{};
    a.s = s;
    a.q = static_cast<const bf16*>(q);
    a.kc = static_cast<const bf16*>(kc);
    a.vc = static_cast<const bf16*>(vc);
    a.out = static_cast<bf16*>(out);
    a.out_pitch = out_pitch;
    a.scale2 = scale * kLog2e;
    a.pos = pos;
    a.slots = slots;
    a.rows = rows;
    a.pos0 = pos0;
    a.part = static_cast<float*>(work);
    return attention_tiles(a, one_sequence, st);
}

}  // namespace zq
