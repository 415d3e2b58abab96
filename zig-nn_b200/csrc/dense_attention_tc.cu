// Prefill attention on the 5th-generation tensor cores: 128 packed query rows (token, head of the group) of one key
// head per CTA against tiles of 64 keys, softmax in f32.
//
//   S = Q K^T   M = 128 rows, N = 64 keys; both operands K-major in shared memory (128-byte swizzle), two accumulators
//               in tensor memory take turns, so the next tile's scores are computed under this tile's softmax;
//   softmax     one thread per row (its row is a tensor-memory lane): no exchange between threads. The running maximum
//               is raised, and the accumulated output rescaled, only when it grows by more than 2^8: until then the
//               weights are taken against the older maximum, which is exact up to rounding;
//   O += P V    P (bf16) goes through shared memory, V is the N operand as it lies in the cache (rows of keys: MN-major).
// Keys and values come in by 2-D tensor copies over the cache, two stages each.
// Roles: warps 0-3 load Q, do the softmax and write the result; warp 4 issues the copies; warp 5 issues the MMAs and
// owns the tensor memory. Every wait is bounded, as in gemm_bf16.cu.
// Keys behind the last one are masked; what the cache holds there must be finite.
#include "dense.h"
#include "tc_common.cuh"

namespace zq {
namespace {

constexpr uint32_t AT_THREADS = 192;
constexpr uint32_t AT_KEYS = 64;
constexpr uint32_t AT_ATOM = AT_KEYS * 128;   // bytes of 64 keys x 64 dimensions
constexpr uint32_t AT_QATOM = 128 * 128;      // 128 rows x 64 dimensions (or keys)
constexpr float kRaise = 8.0f;                // powers of two that the maximum may lag behind

struct AttnTcParams {
    GqaShape s;
    const bf16* q;
    bf16* out;
    uint32_t out_pitch;
    float scale2;          // scale * log2(e)
    const int32_t* slots;
    uint32_t rows, pos0;
    uint32_t dk, dv;       // 64-wide blocks of a key / value row
    uint32_t tmem_cols;
    unsigned int* err;
};

__device__ __forceinline__ void tc_st32(uint32_t taddr, const uint32_t (&r)[32]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,"
        "%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};" ::"r"(taddr),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
        "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]),
        "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]),
        "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
        : "memory");
}
__device__ __forceinline__ void tc_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// Descriptor of a [keys][64 values] tile read with the values as the operand's rows (MN-major, 128-byte swizzle): 64-value
// blocks `block` bytes apart, groups of 8 keys 1024 bytes apart.
__device__ __forceinline__ uint64_t smem_desc_mn_sw128(uint32_t saddr, uint32_t block) {
    uint64_t d = 0;
    d |= (uint64_t)((saddr & 0x3FFFFu) >> 4);
    d |= (uint64_t)(block >> 4) << 16;
    d |= (uint64_t)(1024u >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}

__device__ __forceinline__ uint32_t pack2(float a, float b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&v);
}

__global__ void __launch_bounds__(AT_THREADS, 1)
gqa_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                      const __grid_constant__ AttnTcParams p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ __align__(8) unsigned long long bars[17];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    pdl_launch_dependents();
    const GqaShape& s = p.s;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t base = ((uint32_t)__cvta_generic_to_shared(smem) + 1023u) & ~1023u;
    const uint32_t bar32 = (uint32_t)__cvta_generic_to_shared(bars);
    const uint32_t q_full = bar32;
    auto k_full = [&](uint32_t i) { return bar32 + 8 * (1 + i); };
    auto k_empty = [&](uint32_t i) { return bar32 + 8 * (3 + i); };
    auto v_full = [&](uint32_t i) { return bar32 + 8 * (5 + i); };
    auto v_empty = [&](uint32_t i) { return bar32 + 8 * (7 + i); };
    auto s_full = [&](uint32_t i) { return bar32 + 8 * (9 + i); };
    auto s_empty = [&](uint32_t i) { return bar32 + 8 * (11 + i); };
    auto p_full = [&](uint32_t i) { return bar32 + 8 * (13 + i); };
    auto pv_done = [&](uint32_t i) { return bar32 + 8 * (15 + i); };  // a barrier per P buffer
    // shared memory: Q [dk atoms], K [2][dk atoms], V [2][dv atoms], P [2]
    const uint32_t q_at = base, k_at = q_at + p.dk * AT_QATOM, v_at = k_at + 2 * p.dk * AT_ATOM, p_at = v_at + 2 * p.dv * AT_ATOM;

    const uint32_t R = s.heads / s.kv_heads, g = blockIdx.y, n_rows = p.rows * R;
    const uint32_t m0 = (gridDim.x - 1 - blockIdx.x) * 128;  // the longest tiles first
    const uint32_t last = min(m0 + 128, n_rows) - 1;
    const uint32_t k_end = p.pos0 + last / R + 1, n_tiles = (k_end + AT_KEYS - 1) / AT_KEYS;

    if (tid == 0) {
        mbar_init(q_full, 4);
        for (uint32_t i = 0; i < 2; ++i) {
            mbar_init(k_full(i), 1);
            mbar_init(k_empty(i), 1);
            mbar_init(v_full(i), 1);
            mbar_init(v_empty(i), 1);
            mbar_init(s_full(i), 1);
            mbar_init(s_empty(i), 4);
            mbar_init(p_full(i), 4);
            mbar_init(pv_done(i), 1);
        }
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 5) {
        const uint32_t slot = (uint32_t)__cvta_generic_to_shared(&tmem_slot);
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(slot), "r"(p.tmem_cols)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot, o_col = 2 * AT_KEYS;  // S 0 | S 1 | O
    volatile int* ab = &abort_flag;
    pdl_wait();

    if (warp == 4) {
        if (lane == 0) {
            const uint32_t row0 = (uint32_t)p.slots[0] * s.ctx;
            asm volatile("fence.proxy.async.global;" ::: "memory");
            bool alive = true;
            uint32_t n_k = 0, n_v = 0;  // tiles asked for
            for (uint32_t t = 0; t < n_tiles && alive; ++t) {
                const uint32_t b = t & 1, use = t >> 1;
                if (use > 0) alive = mbar_wait(k_empty(b), (use - 1) & 1u, ab, p.err);
                if (!alive) break;
                mbar_expect_tx(k_full(b), p.dk * AT_ATOM);
                for (uint32_t a = 0; a < p.dk; ++a)
                    tensor_copy_2d(k_at + (b * p.dk + a) * AT_ATOM, &map_k, g * s.dimp * 2 + a * 128, row0 + t * AT_KEYS, k_full(b));
                mbar_arrive(k_full(b));
                ++n_k;
                if (use > 0) alive = mbar_wait(v_empty(b), (use - 1) & 1u, ab, p.err);
                if (!alive) break;
                mbar_expect_tx(v_full(b), p.dv * AT_ATOM);
                for (uint32_t a = 0; a < p.dv; ++a)
                    tensor_copy_2d(v_at + (b * p.dv + a) * AT_ATOM, &map_v, g * s.vdimp * 2 + a * 128, row0 + t * AT_KEYS, v_full(b));
                mbar_arrive(v_full(b));
                ++n_v;
            }
            if (!alive) {  // copies still in flight land before the CTA may retire
                for (uint32_t back = 1; back <= 2; ++back) {
                    for (uint32_t i = 0; back <= n_k && i < kSpinLimit; ++i)
                        if (mbar_try_wait(k_full((n_k - back) & 1), ((n_k - back) >> 1) & 1u)) break;
                    for (uint32_t i = 0; back <= n_v && i < kSpinLimit; ++i)
                        if (mbar_try_wait(v_full((n_v - back) & 1), ((n_v - back) >> 1) & 1u)) break;
                }
            }
        }
        __syncwarp();
    } else if (warp == 5) {
        if (lane == 0) {
            const uint32_t id_s = idesc_bf16(128, AT_KEYS), id_o = idesc_bf16(128, s.vdimp) | (1u << 16);  // V: MN-major
            bool alive = mbar_wait(q_full, 0, ab, p.err);
            auto scores = [&](uint32_t t) {
                const uint32_t b = t & 1, use = t >> 1;
                if (!mbar_wait(k_full(b), use & 1u, ab, p.err)) return false;
                if (use > 0 && !mbar_wait(s_empty(b), (use - 1) & 1u, ab, p.err)) return false;
                tc_fence_after();
                for (uint32_t a = 0; a < p.dk; ++a) {
                    const uint64_t qd = smem_desc_sw128(q_at + a * AT_QATOM), kd = smem_desc_sw128(k_at + (b * p.dk + a) * AT_ATOM);
#pragma unroll
                    for (uint32_t k16 = 0; k16 < 4; ++k16)
                        tc_mma_f16(tmem + b * AT_KEYS, qd + 2 * k16, kd + 2 * k16, id_s, (a | k16) != 0 ? 1u : 0u);
                }
                tc_commit(k_empty(b));
                tc_commit(s_full(b));
                return true;
            };
            if (alive) alive = scores(0);
            for (uint32_t t = 0; t < n_tiles && alive; ++t) {
                const uint32_t b = t & 1, use = t >> 1;
                if (t + 1 < n_tiles) alive = scores(t + 1);
                if (!alive) break;
                alive = mbar_wait(p_full(b), use & 1u, ab, p.err) && mbar_wait(v_full(b), use & 1u, ab, p.err);
                if (!alive) break;
                tc_fence_after();
                const uint64_t pd = smem_desc_sw128(p_at + b * AT_QATOM), vd = smem_desc_mn_sw128(v_at + b * p.dv * AT_ATOM, AT_ATOM);
#pragma unroll
                for (uint32_t k16 = 0; k16 < 4; ++k16)  // 16 keys: 32 bytes of P, two groups of 8 rows of V
                    tc_mma_f16(tmem + o_col, pd + 2 * k16, vd + (2048 >> 4) * k16, id_o, (t | k16) != 0 ? 1u : 0u);
                tc_commit(v_empty(b));
                tc_commit(pv_done(b));
            }
            if (!alive) *ab = 1;
        }
        __syncwarp();
    } else {
        const uint32_t row = m0 + tid;
        const bool real = row < n_rows;
        const uint32_t token = (real ? row : last) / R, head = g * R + (real ? row : last) % R;
        {
            const uint4* src = reinterpret_cast<const uint4*>(p.q + ((size_t)token * s.heads + head) * s.dimp);
            for (uint32_t c = 0; c < p.dk * 8; ++c) {
                const uint4 v = real && c < s.dimp / 8 ? __ldg(src + c) : make_uint4(0, 0, 0, 0);
                const uint32_t at = q_at + (c >> 3) * AT_QATOM + tid * 128u + (((c & 7u) ^ (tid & 7u)) << 4);
                asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};" ::"r"(at), "r"(v.x), "r"(v.y), "r"(v.z), "r"(v.w) : "memory");
            }
            fence_proxy_async();
            __syncwarp();
            if (lane == 0) mbar_arrive(q_full);
        }
        const uint32_t lanes = (warp * 32u) << 16;
        const uint32_t see = real ? p.pos0 + token + 1 : 0;
        float m = -INFINITY, l = 0.0f;
        bool alive = true;
        // O += P V of tile i has finished (a barrier's next phase needs this warp first, so it is never two ahead)
        auto wait_pv = [&](uint32_t i) { alive = __all_sync(0xFFFFFFFFu, mbar_wait(pv_done(i & 1), (i >> 1) & 1u, ab, p.err)); };
        for (uint32_t t = 0; t < n_tiles; ++t) {
            const uint32_t b = t & 1, use = t >> 1, k0 = t * AT_KEYS;
            alive = __all_sync(0xFFFFFFFFu, mbar_wait(s_full(b), use & 1u, ab, p.err));
            if (!alive) break;
            tc_fence_after();
            uint32_t sv[2][32];
            tc_ld32(tmem + lanes + b * AT_KEYS, sv[0]);
            tc_ld32(tmem + lanes + b * AT_KEYS + 32, sv[1]);
            tc_wait_ld();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(s_empty(b));
            float mx = -INFINITY;
            const int lim = (int)see - (int)k0;  // keys of the tile that the row sees
            // scores are scaled on the way into the exponent (a negative scale turns the order round)
            if (p.scale2 <= 0.0f) {
#pragma unroll
                for (int i = 0; i < 64; ++i)
                    if (i < lim) mx = fmaxf(mx, __uint_as_float(sv[i >> 5][i & 31]) * p.scale2);
            } else {
                if (lim >= (int)AT_KEYS) {
#pragma unroll
                    for (int i = 0; i < 64; ++i) mx = fmaxf(mx, __uint_as_float(sv[i >> 5][i & 31]));
                } else {
#pragma unroll
                    for (int i = 0; i < 64; ++i)
                        if (i < lim) mx = fmaxf(mx, __uint_as_float(sv[i >> 5][i & 31]));
                }
                mx *= p.scale2;
            }
            if (t == 0) {
                m = mx;
            } else if (__any_sync(0xFFFFFFFFu, mx - m > kRaise)) {
                const float to = fmaxf(m, mx), f = m == -INFINITY ? 1.0f : exp2f(m - to);
                wait_pv(t - 1);  // O holds tiles 0 .. t - 1
                if (!alive) break;
                tc_fence_after();
                for (uint32_t c = 0; c < s.vdimp; c += 32) {
                    uint32_t o[32];
                    tc_ld32(tmem + lanes + o_col + c, o);
                    tc_wait_ld();
#pragma unroll
                    for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
                    tc_st32(tmem + lanes + o_col + c, o);
                }
                tc_wait_st();
                l *= f;
                m = to;
            }
            const float shift = m == -INFINITY ? 0.0f : m;
            if (t >= 2) wait_pv(t - 2);  // it has read this P buffer
            if (!alive) break;
            const uint32_t prow = p_at + b * AT_QATOM + tid * 128u;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                uint32_t w[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = c * 8 + e * 2;
                    float x = __uint_as_float(sv[i >> 5][i & 31]), y = __uint_as_float(sv[(i + 1) >> 5][(i + 1) & 31]);
                    x = i < lim ? exp2f(fmaf(x, p.scale2, -shift)) : 0.0f;
                    y = i + 1 < lim ? exp2f(fmaf(y, p.scale2, -shift)) : 0.0f;
                    w[e] = pack2(x, y);
                    l += bf16_lo(w[e]) + bf16_hi(w[e]);
                }
                asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};" ::"r"(prow + ((c ^ (tid & 7u)) << 4)), "r"(w[0]), "r"(w[1]),
                             "r"(w[2]), "r"(w[3])
                             : "memory");
            }
            fence_proxy_async();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full(b));
        }
        if (alive) wait_pv(n_tiles - 1);
        if (alive) {
            tc_fence_after();
            bf16* out = p.out + (size_t)token * p.out_pitch + (size_t)head * s.vdim;
            const float inv = 1.0f / l;
            const bool wide = (((uintptr_t)out) & 15u) == 0;
            for (uint32_t c = 0; c < s.vdim; c += 32) {
                uint32_t o[32];
                tc_ld32(tmem + lanes + o_col + c, o);
                tc_wait_ld();
                if (!real) continue;
                if (wide && c + 32 <= s.vdim) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        uint4 w;
                        w.x = pack2(__uint_as_float(o[8 * i]) * inv, __uint_as_float(o[8 * i + 1]) * inv);
                        w.y = pack2(__uint_as_float(o[8 * i + 2]) * inv, __uint_as_float(o[8 * i + 3]) * inv);
                        w.z = pack2(__uint_as_float(o[8 * i + 4]) * inv, __uint_as_float(o[8 * i + 5]) * inv);
                        w.w = pack2(__uint_as_float(o[8 * i + 6]) * inv, __uint_as_float(o[8 * i + 7]) * inv);
                        reinterpret_cast<uint4*>(out + c)[i] = w;
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (c + i < s.vdim) out[c + i] = __float2bfloat16_rn(__uint_as_float(o[i]) * inv);
                }
            }
            if (g == 0 && real && row % R == 0)  // columns beyond the heads
                for (uint32_t i = s.heads * s.vdim; i < p.out_pitch; ++i)
                    p.out[(size_t)token * p.out_pitch + i] = __float2bfloat16_rn(0.0f);
        }
        if (!alive) *ab = 1;
    }

    tc_fence_before();
    __syncthreads();
    if (warp == 5) {
        if (abort_flag && lane == 0) {  // instructions in flight get a bounded chance to finish (gemm_bf16.cu)
            mbar_init(q_full, 1);
            tc_commit(q_full);
            for (uint32_t i = 0; i < kSpinLimit; ++i)
                if (mbar_try_wait(q_full, 0)) break;
        }
        __syncwarp();
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(p.tmem_cols) : "memory");
    }
}

}  // namespace

int launch_gqa_prefill_tc(const GqaShape& s, const bf16* q, const bf16* kc, const bf16* vc, bf16* out, uint32_t out_pitch,
                          float scale2, const int32_t* slots, uint32_t rows, uint32_t pos0, cudaStream_t st) {
    AttnTcParams p{};
    p.s = s;
    p.q = q;
    p.out = out;
    p.out_pitch = out_pitch;
    p.scale2 = scale2;
    p.slots = slots;
    p.rows = rows;
    p.pos0 = pos0;
    p.dk = (s.dimp + 63) / 64;
    p.dv = (s.vdimp + 63) / 64;
    p.tmem_cols = 2 * AT_KEYS + s.vdimp <= 256 ? 256 : 512;
    int rc = device_error_word(&p.err);
    if (rc != ZQ_OK) return rc;
    CUtensorMap mk, mv;
    const uint64_t cache_rows = (uint64_t)s.slots * s.ctx;
    if ((rc = tensor_map_2d(kc, (uint64_t)s.kv_heads * s.dimp * 2, cache_rows, 128, AT_KEYS, 128, &mk)) != ZQ_OK) return rc;
    if ((rc = tensor_map_2d(vc, (uint64_t)s.kv_heads * s.vdimp * 2, cache_rows, 128, AT_KEYS, 128, &mv)) != ZQ_OK) return rc;
    const uint32_t smem = p.dk * AT_QATOM + 2 * (p.dk + p.dv) * AT_ATOM + 2 * AT_QATOM + 1024;
    ZQ_CUDA(cudaFuncSetAttribute(gqa_prefill_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const uint32_t R = s.heads / s.kv_heads;
    const cudaError_t e = launch_pdl(gqa_prefill_tc_kernel, dim3((rows * R + 127) / 128, s.kv_heads), dim3(AT_THREADS), smem, st,
                                     mk, mv, p);
    return e == cudaSuccess ? ZQ_OK : cuda_fail(e);
}

}  // namespace zq
