// Index of the largest logit on the device (greedy decoding of every engine).
#include "zq_internal.h"

namespace zq {
namespace {

// ---- argmax, first maximum wins (src/models/gpt2.zig:980-990) --------------------------------

__device__ __forceinline__ void argmax_merge(float& v, uint32_t& i, float ov, uint32_t oi) {
    if (ov > v || (ov == v && oi < i)) {
        v = ov;
        i = oi;
    }
}

__global__ void __launch_bounds__(1024)
argmax_kernel(const float* __restrict__ logits, uint32_t n, int32_t* __restrict__ out) {
    __shared__ float sv[32];
    __shared__ uint32_t si[32];
    float v = -INFINITY;
    uint32_t idx = 0xFFFFFFFFu;
    // a NaN never compares greater, as in the CPU loop; index 0 is the fallback
    auto take = [&](float c, uint32_t i) {
        if (c > v || (c == v && i < idx)) {
            v = c;
            idx = i;
        }
    };
    uint32_t done = 0;
    if ((reinterpret_cast<uintptr_t>(logits) & 15u) == 0) {
        // four independent 128-bit loads in flight per thread: one CTA reads the row at L2 speed
        const float4* l4 = reinterpret_cast<const float4*>(logits);
        const uint32_t n4 = n / 4, stride = blockDim.x;
        uint32_t i = threadIdx.x;
        for (; i + 3 * stride < n4; i += 4 * stride) {
            float4 c[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) c[u] = __ldg(l4 + i + u * stride);
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const uint32_t b = (i + u * stride) * 4;
                take(c[u].x, b); take(c[u].y, b + 1); take(c[u].z, b + 2); take(c[u].w, b + 3);
            }
        }
        for (; i < n4; i += stride) {
            const float4 c = __ldg(l4 + i);
            take(c.x, i * 4); take(c.y, i * 4 + 1); take(c.z, i * 4 + 2); take(c.w, i * 4 + 3);
        }
        done = n4 * 4;
    }
    for (uint32_t i = done + threadIdx.x; i < n; i += blockDim.x) take(logits[i], i);
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
        const float ov = __shfl_xor_sync(0xFFFFFFFFu, v, off);
        const uint32_t oi = __shfl_xor_sync(0xFFFFFFFFu, idx, off);
        argmax_merge(v, idx, ov, oi);
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (lane == 0) {
        sv[warp] = v;
        si[warp] = idx;
    }
    __syncthreads();
    if (warp == 0) {
        const int nw = blockDim.x >> 5;
        v = lane < nw ? sv[lane] : -INFINITY;
        idx = lane < nw ? si[lane] : 0xFFFFFFFFu;
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) {
            const float ov = __shfl_xor_sync(0xFFFFFFFFu, v, off);
            const uint32_t oi = __shfl_xor_sync(0xFFFFFFFFu, idx, off);
            argmax_merge(v, idx, ov, oi);
        }
        if (lane == 0) out[0] = (idx == 0xFFFFFFFFu) ? 0 : (int32_t)idx;
    }
}

}  // namespace
}  // namespace zq

extern "C" {

int zq_argmax(const float* d_logits, uint32_t n, int32_t* d_index, zq_stream stream) {
    if (!d_logits || !d_index || n == 0) return ZQ_ERR_BAD_ARG;
    zq::argmax_kernel<<<1, 1024, 0, zq::as_stream(stream)>>>(d_logits, n, d_index);
    ZQ_LAUNCH_CHECK();
    return ZQ_OK;
}

}  // extern "C"
