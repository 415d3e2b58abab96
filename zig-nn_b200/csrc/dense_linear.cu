// Linears over bf16 weights for few activation rows: one warp (or, for short deep matrices, the four warps of a
// CTA) per few weight rows, 16-byte weight loads one step ahead of their use, the first of them ahead of the wait
// for the producing kernel. f32 activations take this path for any number of rows; many bf16 rows go to the
// tensor cores (gemm_bf16.cu).
#include "dense.h"

namespace zq {
namespace {

constexpr int kGemvWarps = 4;

struct GemvParams {
    const bf16* w;
    uint32_t kp;
    const void* x;
    uint32_t T;
    void* y;              // f32 outputs, or activation outputs of a GLU
    uint32_t y_stride;
    LinGroups groups;
    GluSpec glu;
    bool prefetch;        // ask L2 for the warp's whole rows while the producing kernel still runs
    // mixture of experts: blockIdx.y = pair (then the tokens of the shared expert)
    const int32_t* ids;
    const float* weights;  // of the pairs' inputs (null: 1)
    uint32_t top, n_pairs, rows_per_expert;
    bool x_by_pair;       // x row = pair (down projection) instead of token
    const bf16* w_shared;
    uint32_t kp_shared, rows_shared;
    const void* x_shared;  // x rows of the shared expert when x_by_pair
    uint32_t y_stride_shared;
    void* y_shared;
    GluSpec glu_shared;
};

// TR activation rows x RW weight rows per warp; SK: the four warps share the rows and split K.
// GLU: RW counts features, each one gate and one up row.
template <typename TX, int TR, int RW, bool SK, bool GLU, bool MOE>
__global__ void __launch_bounds__(kGemvWarps * 32)
dense_gemv_kernel(const __grid_constant__ GemvParams p) {
    constexpr int NR = GLU ? 2 * RW : RW;
    __shared__ float red[SK ? kGemvWarps * NR * TR : 1];
    pdl_launch_dependents();
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const uint32_t j0 = (SK ? blockIdx.x : blockIdx.x * kGemvWarps + warp) * RW;
    const bf16* w = p.w;
    uint32_t kp = p.kp, rows, w_row0, x_row0, y_col = 0, t0 = 0, nt = TR, y_stride = p.y_stride;
    const TX* x = static_cast<const TX*>(p.x);
    void* yv = p.y;
    float in_scale = 1.0f;
    GluSpec glu = p.glu;
    uint32_t pair = 0, y_row0;
    bool waited = false;
    if (MOE) {
        pair = blockIdx.y;
        if (pair < p.n_pairs) {
            pdl_wait();
            waited = true;
            rows = p.rows_per_expert;
            w_row0 = (uint32_t)p.ids[pair] * (GLU ? 2 * rows : rows);
            x_row0 = p.x_by_pair ? pair : pair / p.top;
            if (GLU && p.weights) in_scale = p.weights[pair];
            y_row0 = pair;
        } else {
            const uint32_t t = pair - p.n_pairs;
            w = p.w_shared;
            kp = p.kp_shared;
            rows = p.rows_shared;
            w_row0 = 0;
            if (p.x_by_pair) x = static_cast<const TX*>(p.x_shared);
            x_row0 = t;
            y_row0 = t;
            yv = p.y_shared;
            y_stride = p.y_stride_shared;
            glu = p.glu_shared;
        }
    } else {
        const LinGroup g = p.groups.g[blockIdx.y];
        rows = g.rows;
        w_row0 = g.w_row;
        t0 = blockIdx.z * TR;
        nt = p.T - t0 < (uint32_t)TR ? p.T - t0 : TR;
        x_row0 = g.x_row + t0;
        y_row0 = t0;
        y_col = g.y_col;
    }
    if (j0 >= rows) return;  // uniform over the warp (over the CTA with SK)

    const uint4* wr[NR];
#pragma unroll
    for (int r = 0; r < NR; ++r) {
        const uint32_t j = min(j0 + (GLU ? r / 2 : r), rows - 1);
        const uint32_t row = w_row0 + (GLU ? glu_row(j, r & 1) : j);
        wr[r] = reinterpret_cast<const uint4*>(w + (size_t)row * kp);
    }
    if (!MOE && p.prefetch && lane < NR && (!SK || warp == 0)) {
        const uint32_t j = min(j0 + (GLU ? lane / 2 : lane), rows - 1);
        prefetch_l2_bulk(w + (size_t)(w_row0 + (GLU ? glu_row(j, lane & 1) : j)) * kp, kp * 2);
    }
    const TX* xr[TR];
#pragma unroll
    for (int t = 0; t < TR; ++t) xr[t] = x + (size_t)(x_row0 + min((uint32_t)t, nt - 1)) * kp;

    const uint32_t n_chunks = kp / 8;  // 16 bytes of a weight row each
    const uint32_t step = SK ? kGemvWarps * 32 : 32;
    uint32_t c = SK ? threadIdx.x : lane;
    float acc[NR][TR];
#pragma unroll
    for (int r = 0; r < NR; ++r)
#pragma unroll
        for (int t = 0; t < TR; ++t) acc[r][t] = 0.0f;

    constexpr int U = NR >= 4 ? 1 : (NR == 2 ? 2 : 4);  // chunks held ahead
    uint4 cur[U][NR];
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
        for (int r = 0; r < NR; ++r)
            cur[u][r] = c + u * step < n_chunks ? __ldg(wr[r] + c + u * step) : make_uint4(0, 0, 0, 0);
    if (!waited) pdl_wait();
    while (c < n_chunks) {
        uint4 nxt[U][NR];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const uint32_t cn = c + (U + u) * step;
#pragma unroll
            for (int r = 0; r < NR; ++r) nxt[u][r] = cn < n_chunks ? __ldg(wr[r] + cn) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const uint32_t cc = c + u * step;
            if (cc < n_chunks) {
                float wf[NR][8];
#pragma unroll
                for (int r = 0; r < NR; ++r) unpack8(cur[u][r], wf[r]);
#pragma unroll
                for (int t = 0; t < TR; ++t) {
                    float xf[8];
                    load8(xr[t] + (size_t)cc * 8, xf);
#pragma unroll
                    for (int r = 0; r < NR; ++r)
#pragma unroll
                        for (int e = 0; e < 8; ++e) acc[r][t] = fmaf(wf[r][e], xf[e], acc[r][t]);
                }
            }
        }
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int r = 0; r < NR; ++r) cur[u][r] = nxt[u][r];
        c += U * step;
    }
#pragma unroll
    for (int r = 0; r < NR; ++r)
#pragma unroll
        for (int t = 0; t < TR; ++t) acc[r][t] = warp_sum_f(acc[r][t]);
    if (SK) {
        if (lane == 0) {
#pragma unroll
            for (int r = 0; r < NR; ++r)
#pragma unroll
                for (int t = 0; t < TR; ++t) red[(warp * NR + r) * TR + t] = acc[r][t];
        }
        __syncthreads();
        if (warp != 0) return;
#pragma unroll
        for (int r = 0; r < NR; ++r)
#pragma unroll
            for (int t = 0; t < TR; ++t) {
                float s = red[r * TR + t];
#pragma unroll
                for (int q = 1; q < kGemvWarps; ++q) s += red[(q * NR + r) * TR + t];
                acc[r][t] = s;
            }
    }
    // the values of the warp are the same in every lane: lane i writes value i
#pragma unroll
    for (int f = 0; f < RW; ++f)
#pragma unroll
        for (int t = 0; t < TR; ++t) {
            if (lane != (uint32_t)((f * TR + t) & 31) || j0 + f >= rows || (uint32_t)t >= nt) continue;
            const size_t o = (size_t)(y_row0 + t) * y_stride + y_col + j0 + f;
            if (GLU)
                static_cast<TX*>(yv)[o] = to_act<TX>(
                    glu_value(acc[2 * f][t] * in_scale, acc[(2 * f + 1) % NR][t] * in_scale, glu.kind, glu.limit));
            else
                static_cast<float*>(yv)[o] = acc[f][t];
        }
}

template <typename TX, int TR, bool GLU, bool MOE>
int gemv_shape(GemvParams p, uint32_t rows, uint32_t kp, uint32_t gy, uint32_t gz, cudaStream_t st) {
    p.prefetch = (uint64_t)rows * (GLU ? 2 : 1) * gy * kp * 2 <= (64u << 20);  // a part of L2 at most
    // Two rows (features) per warp when there are warps enough to fill the GPU that way, the K split when one row
    // per warp does not.
    const uint64_t per_sm = (uint64_t)sm_count() * 16;
    const uint64_t total = (uint64_t)rows * gy * gz;
    cudaError_t e;
    if (total >= 2 * per_sm) {
        e = launch_pdl(dense_gemv_kernel<TX, TR, 2, false, GLU, MOE>, dim3((rows + 2 * kGemvWarps - 1) / (2 * kGemvWarps), gy, gz),
                       dim3(kGemvWarps * 32), 0, st, p);
    } else if (total < per_sm && kp >= 1024) {
        e = launch_pdl(dense_gemv_kernel<TX, TR, 1, true, GLU, MOE>, dim3(rows, gy, gz), dim3(kGemvWarps * 32), 0, st, p);
    } else {
        e = launch_pdl(dense_gemv_kernel<TX, TR, 1, false, GLU, MOE>, dim3((rows + kGemvWarps - 1) / kGemvWarps, gy, gz),
                       dim3(kGemvWarps * 32), 0, st, p);
    }
    if (e != cudaSuccess) return cuda_fail(e);
    return ZQ_OK;
}

template <typename TX, bool GLU>
int gemv_rows(const GemvParams& p, uint32_t rows, uint32_t n_groups, cudaStream_t st) {
    if (p.T == 1) return gemv_shape<TX, 1, GLU, false>(p, rows, p.kp, n_groups, 1, st);
    if (p.T == 2) return gemv_shape<TX, 2, GLU, false>(p, rows, p.kp, n_groups, 1, st);
    if (p.T <= 4) return gemv_shape<TX, 4, GLU, false>(p, rows, p.kp, n_groups, 1, st);
    return gemv_shape<TX, 8, GLU, false>(p, rows, p.kp, n_groups, (p.T + 7) / 8, st);
}

}  // namespace

int launch_dense_linear(const DenseWeight& W, const LinGroups& G, const void* x, uint32_t x_rows, uint32_t T, float* y,
                        uint32_t y_stride, bool f32, cudaStream_t st, Addends* add, size_t y_floats) {
    if (add) *add = Addends{};
    if (T == 0) return ZQ_OK;
    if (!f32 && T >= kDenseGemmMinRows)
        return launch_gemm_bf16(W, G, static_cast<const bf16*>(x), x_rows, T, y, y_stride, nullptr, 0, nullptr, st, add,
                                y_floats);
    GemvParams p{};
    p.w = W.w;
    p.kp = W.kp;
    p.x = x;
    p.T = T;
    p.y = y;
    p.y_stride = y_stride;
    p.groups = G;
    uint32_t rows = 0;
    for (uint32_t i = 0; i < G.n; ++i) rows = rows > G.g[i].rows ? rows : G.g[i].rows;
    return f32 ? gemv_rows<float, false>(p, rows, G.n, st) : gemv_rows<bf16, false>(p, rows, G.n, st);
}

int launch_dense_glu(const DenseWeight& W, const void* x, uint32_t T, void* out, GluSpec glu, bool f32, cudaStream_t st) {
    if (T == 0) return ZQ_OK;
    const uint32_t ffp = W.rows / 2;
    if (!f32 && T >= kDenseGemmMinRows)
        return launch_gemm_bf16(W, one_group(W.rows), static_cast<const bf16*>(x), T, T, nullptr, 0, static_cast<bf16*>(out),
                                ffp, &glu, st);
    GemvParams p{};
    p.w = W.w;
    p.kp = W.kp;
    p.x = x;
    p.T = T;
    p.y = out;
    p.y_stride = ffp;
    p.groups = one_group(ffp);
    p.glu = glu;
    return f32 ? gemv_rows<float, true>(p, ffp, 1, st) : gemv_rows<bf16, true>(p, ffp, 1, st);
}

int launch_moe_pairs(const MoeWeights& M, const MoeRouting& R, const void* x, uint32_t T, void* hidden, float* parts,
                     bool f32, cudaStream_t st) {
    if (T == 0) return ZQ_OK;
    const uint32_t pairs = T * M.top, gy = pairs + (M.shared_ffp ? T : 0);
    if (gy > 65535) return ZQ_ERR_LIMIT;
    GemvParams p{};
    p.ids = R.ids;
    p.weights = M.scale_input ? R.weights : nullptr;
    p.top = M.top;
    p.n_pairs = pairs;
    // gate | up of every pair
    p.w = M.gate_up.w;
    p.kp = M.gate_up.kp;
    p.x = x;
    p.y = hidden;
    p.y_stride = M.ffp;
    p.rows_per_expert = M.ffp;
    p.glu = M.glu;
    p.glu_shared = M.shared_glu;
    p.w_shared = M.shared_gate_up.w;
    p.kp_shared = M.shared_gate_up.kp;
    p.rows_shared = M.shared_ffp;
    p.y_stride_shared = M.shared_ffp;
    void* hidden_shared = static_cast<char*>(hidden) + (size_t)pairs * M.ffp * act_bytes(f32);
    p.y_shared = hidden_shared;
    const uint32_t rows = M.ffp > M.shared_ffp ? M.ffp : M.shared_ffp;
    int rc = f32 ? gemv_shape<float, 1, true, true>(p, rows, p.kp, gy, 1, st)
                 : gemv_shape<bf16, 1, true, true>(p, rows, p.kp, gy, 1, st);
    if (rc != ZQ_OK) return rc;
    // down
    p.w = M.down.w;
    p.kp = M.down.kp;
    p.x = hidden;
    p.x_by_pair = true;
    p.x_shared = hidden_shared;
    p.y = parts;
    p.y_stride = M.width;
    p.rows_per_expert = M.width;
    p.w_shared = M.shared_down.w;
    p.kp_shared = M.shared_down.kp;
    p.rows_shared = M.width;
    p.y_shared = parts + (size_t)pairs * M.width;
    p.y_stride_shared = M.width;
    return f32 ? gemv_shape<float, 1, false, true>(p, M.width, p.kp, gy, 1, st)
               : gemv_shape<bf16, 1, false, true>(p, M.width, p.kp, gy, 1, st);
}

}  // namespace zq
