// Row-wise steps between the products of a bf16-weight decoder: embedding, norms with the residual sum, token shift,
// query / key norms with the cache write, and the routing of a mixture of experts. Everything is computed in f32.
#include "dense.h"

namespace zq {
namespace {

// ---- residual sum + next norm (+ token shift) -----------------------------------------------------------------
template <typename TA>
__global__ void __launch_bounds__(256)
add_norm_kernel(const __grid_constant__ AddNormArgs a) {
    extern __shared__ __align__(16) float row[];  // the residual row, later h
    __shared__ float red[33];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t r = blockIdx.x, W = a.width;
    const uint32_t src = a.rows_from ? (uint32_t)a.rows_from[r] : r;
    float* x = a.x + (size_t)src * W;
    if (a.embed) {
        const bf16* e = a.embed + (size_t)a.tokens[r] * a.embed_kp;
        for (uint32_t i = threadIdx.x; i < W; i += blockDim.x) {
            const float v = __bfloat162float(e[i]) * a.embed_scale;
            row[i] = v;
            if (!a.embed_w) x[i] = v;
        }
        if (a.embed_w) {  // every thread reads back what it wrote
            float ss = 0.0f;
            for (uint32_t i = threadIdx.x; i < W; i += blockDim.x) ss = fmaf(row[i], row[i], ss);
            const float inv = 1.0f / sqrtf(block_sum_f(ss, red) / (float)W + a.eps);
            for (uint32_t i = threadIdx.x; i < W; i += blockDim.x) x[i] = row[i] = row[i] * inv * a.embed_w[i];
        }
    } else if (a.y || a.y2 || a.parts) {
        const float gate = a.shared ? (a.shared_gate ? sigmoid_f(a.shared_gate[(size_t)r * a.gate_stride]) : 1.0f) : 0.0f;
        float ss = 0.0f;
        for (uint32_t i = threadIdx.x; i < W; i += blockDim.x) {
            float v = 0.0f;
            if (a.y)
                for (uint32_t q = 0; q < a.y_add.n; ++q) v += a.y[q * a.y_add.stride + (size_t)r * W + i];
            if (a.y2)
                for (uint32_t q = 0; q < a.y2_add.n; ++q) v += a.y2[q * a.y2_add.stride + (size_t)r * W + i];
            if (a.parts) {
                for (uint32_t k = 0; k < a.top; ++k) {
                    const uint32_t pair = r * a.top + k;
                    const float part = a.parts[(size_t)(a.place ? (uint32_t)a.place[pair] : pair) * W + i];
                    v = a.part_w ? fmaf(a.part_w[pair], part, v) : v + part;
                }
                if (a.shared) v += gate * a.shared[(size_t)r * W + i];
            }
            row[i] = v;
            ss = fmaf(v, v, ss);
        }
        float inv = 1.0f;
        if (a.post_w) inv = 1.0f / sqrtf(block_sum_f(ss, red) / (float)W + a.eps);
        for (uint32_t i = threadIdx.x; i < W; i += blockDim.x) {
            const float v = x[i] + row[i] * inv * (a.post_w ? a.post_w[i] : 1.0f);
            row[i] = v;
            x[i] = v;
        }
    } else {
        for (uint32_t i = threadIdx.x; i < W; i += blockDim.x) row[i] = x[i];
    }
    if (!a.pre_w) return;
    float ss = 0.0f;
    for (uint32_t i = threadIdx.x; i < W; i += blockDim.x) ss = fmaf(row[i], row[i], ss);
    ss = block_sum_f(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)W + a.eps);
    TA* h = static_cast<TA*>(a.h);
    for (uint32_t i = threadIdx.x; i < a.hp; i += blockDim.x) {
        const float v = i < W ? row[i] * inv * a.pre_w[i] : 0.0f;
        if (h) h[(size_t)r * a.hp + i] = to_act<TA>(v);
        if (i >= W) continue;
        if (a.h32) a.h32[(size_t)r * W + i] = v;
        row[i] = v;
    }
    if (!a.n_mix) return;
    float* prev = a.prev + (size_t)a.slots[r] * W;
    TA* mix = static_cast<TA*>(a.mix);
    for (uint32_t i = threadIdx.x; i < a.hp; i += blockDim.x) {  // every thread reads back what it wrote
        const float v = i < W ? row[i] : 0.0f, d = i < W ? prev[i] - v : 0.0f;
        for (uint32_t s = 0; s < a.n_mix; ++s)
            mix[((size_t)s * a.mix_rows + r) * a.hp + i] = to_act<TA>(i < W ? fmaf(d, a.mu[(size_t)s * W + i], v) : 0.0f);
        if (i < W) prev[i] = v;
    }
}

template <typename TA>
__global__ void __launch_bounds__(256)
token_shift_kernel(const float* __restrict__ h32, const float* __restrict__ mu, const float* __restrict__ prev,
                   const int32_t* __restrict__ slots, uint32_t n_mix, uint32_t mix_rows, uint32_t width, uint32_t hp,
                   TA* __restrict__ mix) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t r = blockIdx.x;
    const float* h = h32 + (size_t)r * width;
    const float* before = r ? h - width : prev + (size_t)slots[0] * width;
    for (uint32_t i = threadIdx.x; i < hp; i += blockDim.x) {
        const float v = i < width ? h[i] : 0.0f, d = i < width ? before[i] - v : 0.0f;
        for (uint32_t s = 0; s < n_mix; ++s)
            mix[((size_t)s * mix_rows + r) * hp + i] = to_act<TA>(i < width ? fmaf(d, mu[(size_t)s * width + i], v) : 0.0f);
    }
}

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(bf16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ void add4(float4& a, const float4& b) { a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w; }
__device__ __forceinline__ float sumsq4(const float4& a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }
__device__ __forceinline__ void fma4(float4& a, float f, const float4& b) {
    a.x = fmaf(f, b.x, a.x); a.y = fmaf(f, b.y, a.y); a.z = fmaf(f, b.z, a.z); a.w = fmaf(f, b.w, a.w);
}
__device__ __forceinline__ float4 scaled(const float4& v, float f, const float4& w) {  // v * f * w
    return make_float4(v.x * f * w.x, v.y * f * w.y, v.z * f * w.z, v.w * f * w.w);
}
__device__ __forceinline__ float4 toward(const float4& v, const float4& d, const float4& mu) {  // v + d * mu
    return make_float4(fmaf(d.x, mu.x, v.x), fmaf(d.y, mu.y, v.y), fmaf(d.z, mu.z, v.z), fmaf(d.w, mu.w, v.w));
}

// The same for widths that are multiples of 4: a thread keeps NV float4 of the row in registers, everything that a step
// needs is requested up front (the weights ahead of the wait for the producing kernel).
template <typename TA, int NV>
__global__ void __launch_bounds__(1024)
add_norm_vec_kernel(const __grid_constant__ AddNormArgs a) {
    __shared__ float red[33];
    pdl_launch_dependents();
    const uint32_t r = blockIdx.x, W = a.width, n4 = W / 4, tid = threadIdx.x, nthr = blockDim.x;
    const bool adds = a.y || a.y2 || a.parts;
    const float* first_w = a.embed ? a.embed_w : adds ? a.post_w : nullptr;
    float4 post[NV], pre[NV], x[NV], y[NV];
#pragma unroll
    for (int v = 0; v < NV; ++v) {
        const uint32_t i = tid + v * nthr;
        const bool in = i < n4;
        post[v] = in && first_w ? ld4(first_w + 4 * i) : make_float4(1, 1, 1, 1);
        pre[v] = in && a.pre_w ? ld4(a.pre_w + 4 * i) : make_float4(0, 0, 0, 0);
    }
    pdl_wait();
    const uint32_t src = a.rows_from ? (uint32_t)a.rows_from[r] : r;
    float* xrow = a.x + (size_t)src * W;
    if (a.embed) {
        const bf16* e = a.embed + (size_t)a.tokens[r] * a.embed_kp;
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const uint32_t i = tid + v * nthr;
            x[v] = make_float4(0, 0, 0, 0);
            if (i >= n4) continue;
            const uint2 u = *reinterpret_cast<const uint2*>(e + 4 * i);
            x[v] = make_float4(bf16_lo(u.x) * a.embed_scale, bf16_hi(u.x) * a.embed_scale, bf16_lo(u.y) * a.embed_scale,
                               bf16_hi(u.y) * a.embed_scale);
            if (!a.embed_w) st4(xrow + 4 * i, x[v]);
        }
        if (a.embed_w) {
            float ss = 0.0f;
#pragma unroll
            for (int v = 0; v < NV; ++v) ss += sumsq4(x[v]);
            const float inv = 1.0f / sqrtf(block_sum_f(ss, red) / (float)W + a.eps);
#pragma unroll
            for (int v = 0; v < NV; ++v) {
                const uint32_t i = tid + v * nthr;
                x[v] = scaled(x[v], inv, post[v]);
                if (i < n4) st4(xrow + 4 * i, x[v]);
            }
        }
    } else {
        const float gate = a.shared ? (a.shared_gate ? sigmoid_f(a.shared_gate[(size_t)r * a.gate_stride]) : 1.0f) : 0.0f;
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const uint32_t i = tid + v * nthr;
            x[v] = y[v] = make_float4(0, 0, 0, 0);
            if (i >= n4) continue;
            x[v] = ld4(xrow + 4 * i);
            if (a.y) {
                const float* p = a.y + (size_t)r * W + 4 * i;
                y[v] = ld4(p);
                for (uint32_t q = 1; q < a.y_add.n; ++q) add4(y[v], ld4(p + q * a.y_add.stride));
            }
            if (a.y2) {
                const float* p = a.y2 + (size_t)r * W + 4 * i;
                for (uint32_t q = 0; q < a.y2_add.n; ++q) add4(y[v], ld4(p + q * a.y2_add.stride));
            }
            if (a.parts) {
                for (uint32_t k = 0; k < a.top; ++k) {
                    const uint32_t pair = r * a.top + k;
                    const float4 part = ld4(a.parts + (size_t)(a.place ? (uint32_t)a.place[pair] : pair) * W + 4 * i);
                    fma4(y[v], a.part_w ? a.part_w[pair] : 1.0f, part);
                }
                if (a.shared) {
                    const float4 s = ld4(a.shared + (size_t)r * W + 4 * i);
                    add4(y[v], make_float4(gate * s.x, gate * s.y, gate * s.z, gate * s.w));
                }
            }
        }
        if (adds) {
            float ss = 0.0f, inv = 1.0f;
#pragma unroll
            for (int v = 0; v < NV; ++v) ss += sumsq4(y[v]);
            if (a.post_w) inv = 1.0f / sqrtf(block_sum_f(ss, red) / (float)W + a.eps);
#pragma unroll
            for (int v = 0; v < NV; ++v) {
                const uint32_t i = tid + v * nthr;
                add4(x[v], scaled(y[v], inv, post[v]));
                if (i < n4) st4(xrow + 4 * i, x[v]);
            }
        }
    }
    if (!a.pre_w) return;
    float4 prev[NV];
    if (a.n_mix) {
        const float* p = a.prev + (size_t)a.slots[r] * W;
#pragma unroll
        for (int v = 0; v < NV; ++v) prev[v] = tid + v * nthr < n4 ? ld4(p + 4 * (tid + v * nthr)) : make_float4(0, 0, 0, 0);
    }
    float ss = 0.0f;
#pragma unroll
    for (int v = 0; v < NV; ++v) ss += sumsq4(x[v]);
    const float inv = 1.0f / sqrtf(block_sum_f(ss, red) / (float)W + a.eps);
    TA* h = a.h ? static_cast<TA*>(a.h) + (size_t)r * a.hp : nullptr;
    TA* mix = a.n_mix ? static_cast<TA*>(a.mix) + (size_t)r * a.hp : nullptr;
#pragma unroll
    for (int v = 0; v < NV; ++v) {
        const uint32_t i = tid + v * nthr;
        if (i >= n4) continue;
        const float4 o = scaled(x[v], inv, pre[v]);
        if (h) st4(h + 4 * i, o);
        if (a.h32) st4(a.h32 + (size_t)r * W + 4 * i, o);
        if (!mix) continue;
        const float4 d = make_float4(prev[v].x - o.x, prev[v].y - o.y, prev[v].z - o.z, prev[v].w - o.w);
        for (uint32_t s = 0; s < a.n_mix; ++s)
            st4(mix + (size_t)s * a.mix_rows * a.hp + 4 * i, toward(o, d, ld4(a.mu + (size_t)s * W + 4 * i)));
        st4(a.prev + (size_t)a.slots[r] * W + 4 * i, o);
    }
    for (uint32_t i = n4 + tid; i < a.hp / 4; i += nthr) {  // columns beyond the width
        if (h) st4(h + 4 * i, make_float4(0, 0, 0, 0));
        for (uint32_t s = 0; mix && s < a.n_mix; ++s) st4(mix + (size_t)s * a.mix_rows * a.hp + 4 * i, make_float4(0, 0, 0, 0));
    }
}

template <typename TA>
__global__ void __launch_bounds__(256)
token_shift_vec_kernel(const float* __restrict__ h32, const float* __restrict__ mu, const float* __restrict__ prev,
                       const int32_t* __restrict__ slots, uint32_t n_mix, uint32_t mix_rows, uint32_t width, uint32_t hp,
                       TA* __restrict__ mix) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t r = blockIdx.x;
    const float* h = h32 + (size_t)r * width;
    const float* before = r ? h - width : prev + (size_t)slots[0] * width;
    for (uint32_t i = threadIdx.x * 4; i < hp; i += blockDim.x * 4) {
        const bool in = i < width;
        const float4 v = in ? ld4(h + i) : make_float4(0, 0, 0, 0), b = in ? ld4(before + i) : v;
        const float4 d = make_float4(b.x - v.x, b.y - v.y, b.z - v.z, b.w - v.w);
        for (uint32_t s = 0; s < n_mix; ++s)
            st4(mix + ((size_t)s * mix_rows + r) * hp + i, in ? toward(v, d, ld4(mu + (size_t)s * width + i)) : v);
    }
}

// ---- q / k norm, query temperature, value mixing, cache write: one warp per head ---------------------------------
template <typename TA>
__global__ void __launch_bounds__(128)
qkv_post_kernel(const __grid_constant__ QkvPostArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const GqaShape& s = a.s;
    const uint32_t lane = threadIdx.x & 31, item = blockIdx.y * 4 + (threadIdx.x >> 5), r = blockIdx.x;
    if (item >= s.heads + 2 * s.kv_heads) return;
    const uint32_t ld = (s.heads + s.kv_heads) * s.dim + s.kv_heads * s.vdim;
    const float* row = a.qkv + (size_t)r * ld;
    const uint32_t pos = (uint32_t)a.pos[r];
    const size_t at = (size_t)(uint32_t)a.slots[r] * s.ctx + pos;
    if (item < s.heads + s.kv_heads) {
        const bool is_q = item < s.heads;
        const float t = is_q ? query_temperature(pos, a.temp_coef, a.temp_every) : 1.0f;
        TA* o = is_q ? static_cast<TA*>(a.q) + ((size_t)r * s.heads + item) * s.dimp
                     : static_cast<TA*>(a.kc) + (at * s.kv_heads + (item - s.heads)) * s.dimp;
        norm_head(row + (size_t)item * s.dim, is_q ? a.q_norm : a.k_norm, s.dim, s.dimp, a.eps, t, o, lane);
    } else {
        const uint32_t g = item - s.heads - s.kv_heads;
        const float* v = row + (size_t)(s.heads + s.kv_heads) * s.dim + (size_t)g * s.vdim;
        float* first = a.v_first ? a.v_first + ((size_t)r * s.kv_heads + g) * s.vdim : nullptr;
        TA* o = static_cast<TA*>(a.vc) + (at * s.kv_heads + g) * s.vdimp;
        for (uint32_t i = lane; i < s.vdimp; i += 32) o[i] = to_act<TA>(i < s.vdim ? mixed_value(v[i], a.vmix, first, i) : 0.0f);
    }
}

// ---- routing ----------------------------------------------------------------------------------------------------
constexpr uint32_t kMaxExperts = 1024;

// One warp per token: the `top` largest logits (the sigmoid keeps their order), lowest id among equal ones; they come out
// in descending order, so the first one is the maximum of the softmax over them.
__global__ void __launch_bounds__(32)
route_kernel(const float* __restrict__ z, uint32_t z_stride, uint32_t experts, uint32_t top, const float* __restrict__ bias,
             int kind, int32_t* __restrict__ ids, float* __restrict__ weights) {
    __shared__ float v[kMaxExperts];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t lane = threadIdx.x, r = blockIdx.x;
    for (uint32_t e = lane; e < experts; e += 32) v[e] = z[(size_t)r * z_stride + e] + (bias ? bias[e] : 0.0f);
    __syncwarp();
    float first = 0.0f, sum = 0.0f;
    for (uint32_t k = 0; k < top; ++k) {
        float best = -INFINITY;
        uint32_t id = 0xFFFFFFFFu;
        for (uint32_t e = lane; e < experts; e += 32)
            if (v[e] > best || id == 0xFFFFFFFFu) {
                best = v[e];
                id = e;
            }
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) {
            const float ob = __shfl_xor_sync(0xFFFFFFFFu, best, off);
            const uint32_t oi = __shfl_xor_sync(0xFFFFFFFFu, id, off);
            if (oi != 0xFFFFFFFFu && (id == 0xFFFFFFFFu || ob > best || (ob == best && oi < id))) {
                best = ob;
                id = oi;
            }
        }
        if (lane == 0) {
            ids[(size_t)r * top + k] = (int32_t)id;
            if (k == 0) first = best;
            const float w = kind == ROUTE_SOFTMAX ? expf(best - first) : sigmoid_f(best);
            sum += w;
            weights[(size_t)r * top + k] = w;
            v[id] = -INFINITY;
        }
        __syncwarp();
    }
    if (kind == ROUTE_SOFTMAX && lane == 0)
        for (uint32_t k = 0; k < top; ++k) weights[(size_t)r * top + k] /= sum;
}

// Counts, offsets, tiles and places of all pairs: one CTA. The order inside an expert is of no consequence.
__global__ void __launch_bounds__(1024)
moe_plan_kernel(const int32_t* __restrict__ ids, uint32_t pairs, uint32_t experts, uint32_t bn, int32_t* __restrict__ place,
                int32_t* __restrict__ source, int32_t* __restrict__ offsets, int32_t* __restrict__ tiles) {
    __shared__ uint32_t count[kMaxExperts], start[kMaxExperts + 1], tile0[kMaxExperts + 1];
    pdl_launch_dependents();
    pdl_wait();
    for (uint32_t e = threadIdx.x; e < experts; e += blockDim.x) count[e] = 0;
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < pairs; i += blockDim.x) atomicAdd(&count[ids[i]], 1u);
    __syncthreads();
    if (threadIdx.x == 0) {
        uint32_t s = 0, t = 0;
        for (uint32_t e = 0; e < experts; ++e) {
            start[e] = s;
            tile0[e] = t;
            s += count[e];
            t += (count[e] + bn - 1) / bn;
        }
        start[experts] = s;
        tile0[experts] = t;
        tiles[0] = (int32_t)t;
    }
    __syncthreads();
    for (uint32_t e = threadIdx.x; e < experts; e += blockDim.x) {
        offsets[e] = (int32_t)start[e];
        for (uint32_t t = tile0[e]; t < tile0[e + 1]; ++t) {
            tiles[1 + 2 * t] = (int32_t)e;
            tiles[2 + 2 * t] = (int32_t)(start[e] + (t - tile0[e]) * bn);
        }
        count[e] = start[e];
    }
    if (threadIdx.x == 0) offsets[experts] = (int32_t)start[experts];
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < pairs; i += blockDim.x) {
        const uint32_t at = atomicAdd(&count[ids[i]], 1u);
        place[i] = (int32_t)at;
        source[at] = (int32_t)i;
    }
}

// xs[row] = h[token of the pair at that row] (times its weight)
__global__ void __launch_bounds__(128)
moe_scatter_kernel(const int32_t* __restrict__ source, const float* __restrict__ weights, const bf16* __restrict__ h,
                   uint32_t top, uint32_t hp, bf16* __restrict__ xs) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t pair = (uint32_t)source[blockIdx.x];
    const float w = weights ? weights[pair] : 1.0f;
    const uint4* src = reinterpret_cast<const uint4*>(h + (size_t)(pair / top) * hp);
    uint4* dst = reinterpret_cast<uint4*>(xs + (size_t)blockIdx.x * hp);
    for (uint32_t c = threadIdx.x; c < hp / 8; c += blockDim.x) {
        float f[8];
        unpack8(src[c], f);
        uint32_t o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(f[2 * e] * w, f[2 * e + 1] * w);
            o[e] = *reinterpret_cast<const uint32_t*>(&b);
        }
        dst[c] = make_uint4(o[0], o[1], o[2], o[3]);
    }
}

int done(cudaError_t e) { return e == cudaSuccess ? ZQ_OK : cuda_fail(e); }

}  // namespace

int launch_add_norm(const AddNormArgs& a, uint32_t rows, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    if (a.width > 12288) return ZQ_ERR_LIMIT;  // the row lies in shared memory
    if (a.width % 4 == 0) {
        const uint32_t n4 = a.width / 4, nv = n4 <= 512 ? 1 : n4 <= 2048 ? 2 : 3;
        const dim3 block(pad_to((n4 + nv - 1) / nv, 32));
        auto go = [&](auto kern) { return done(launch_pdl(kern, dim3(rows), block, 0, st, a)); };
        if (nv == 1) return f32 ? go(add_norm_vec_kernel<float, 1>) : go(add_norm_vec_kernel<bf16, 1>);
        if (nv == 2) return f32 ? go(add_norm_vec_kernel<float, 2>) : go(add_norm_vec_kernel<bf16, 2>);
        return f32 ? go(add_norm_vec_kernel<float, 3>) : go(add_norm_vec_kernel<bf16, 3>);
    }
    const size_t smem = (size_t)a.width * sizeof(float);
    return done(f32 ? launch_pdl(add_norm_kernel<float>, dim3(rows), dim3(256), smem, st, a)
                    : launch_pdl(add_norm_kernel<bf16>, dim3(rows), dim3(256), smem, st, a));
}

int launch_token_shift(const float* h32, const float* mu, const float* prev, const int32_t* slots, uint32_t n_mix,
                       uint32_t rows, uint32_t mix_rows, uint32_t width, void* mix, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    const uint32_t hp = pad64(width);
    if (width % 4 == 0) {
        auto go = [&](auto kern, auto* out) {
            return done(launch_pdl(kern, dim3(rows), dim3(256), 0, st, h32, mu, prev, slots, n_mix, mix_rows, width, hp, out));
        };
        return f32 ? go(token_shift_vec_kernel<float>, static_cast<float*>(mix)) : go(token_shift_vec_kernel<bf16>, static_cast<bf16*>(mix));
    }
    return done(f32 ? launch_pdl(token_shift_kernel<float>, dim3(rows), dim3(256), 0, st, h32, mu, prev, slots, n_mix, mix_rows,
                                 width, hp, static_cast<float*>(mix))
                    : launch_pdl(token_shift_kernel<bf16>, dim3(rows), dim3(256), 0, st, h32, mu, prev, slots, n_mix, mix_rows,
                                 width, hp, static_cast<bf16*>(mix)));
}

int launch_qkv_post(const QkvPostArgs& a, uint32_t rows, bool f32, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    const dim3 grid(rows, (a.s.heads + 2 * a.s.kv_heads + 3) / 4);
    return done(f32 ? launch_pdl(qkv_post_kernel<float>, grid, dim3(128), 0, st, a)
                    : launch_pdl(qkv_post_kernel<bf16>, grid, dim3(128), 0, st, a));
}

int launch_route(const float* z, uint32_t z_stride, uint32_t experts, uint32_t top, const float* bias, int kind,
                 const MoeRouting& R, uint32_t rows, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    if (experts > kMaxExperts || top > experts) return ZQ_ERR_LIMIT;
    return done(launch_pdl(route_kernel, dim3(rows), dim3(32), 0, st, z, z_stride, experts, top, bias, kind, R.ids, R.weights));
}

int launch_moe_plan(const MoeRouting& R, uint32_t experts, uint32_t top, uint32_t rows, uint32_t bn, const bf16* h,
                    uint32_t hp, bool scale_input, bf16* xs, cudaStream_t st) {
    if (rows == 0) return ZQ_OK;
    const uint32_t pairs = rows * top;
    if (experts > kMaxExperts || pairs / bn + experts > kMoeMaxTiles) return ZQ_ERR_LIMIT;
    int rc = done(launch_pdl(moe_plan_kernel, dim3(1), dim3(1024), 0, st, R.ids, pairs, experts, bn, R.place, R.source,
                             R.offsets, R.tiles));
    if (rc != ZQ_OK) return rc;
    const float* weights = scale_input ? R.weights : nullptr;
    return done(launch_pdl(moe_scatter_kernel, dim3(pairs), dim3(128), 0, st, R.source, weights, h, top, hp, xs));
}

}  // namespace zq
