// bf16 x bf16 products on the 5th-generation tensor cores for many activation rows.
//
// A operand (M = 128): 128 weight rows x 64 K per stage; B operand (N up to 256): activation rows x 64 K. Both come
// in by 2-D tensor copies with the 128-byte swizzle; D = 128 lanes (one per weight row) x N columns of f32 in tensor
// memory, two of them taking turns. The kernel is persistent: CTA b walks the tiles b, b + grid, ...
// Roles: warp 0 issues the copies, warp 1 issues the MMAs and owns the tensor memory, warps 2-9 drain a finished
// accumulator (lane quarter warp % 4, column half (warp - 2) / 4) while the next tile's stages flow.
// A launch holds one product, several with their own weight and activation rows (the projections behind a token
// shift), or the experts of a routed batch (tiles listed in device memory).
// Epilogues: f32 out, or the gated unit of an interleaved gate | up weight (16 gate rows and the 16 up rows of the same
// features share a warp: one shuffle brings them together), bf16 out, or bf16 out head by head to two arrays.
// Every wait is bounded; on a timeout the kernel records it, all roles leave their loops, the copies in flight are
// waited for (bounded) and the tensor memory is released.
#include "dense.h"
#include "tc_common.cuh"

namespace zq {
namespace {

constexpr uint32_t GB_THREADS = 320;
constexpr uint32_t GB_EPI_WARPS = 8;
constexpr uint32_t GB_A_BYTES = 128 * 128;
constexpr uint32_t GB_MAX_STAGES = 8;
constexpr uint32_t GB_SMEM = 208 * 1024;  // ring, less than the 227 KB a CTA may have

struct GemmParams {
    uint32_t n_k;        // 64-K stages
    uint32_t k_parts;    // the K dimension cut into that many runs of k_len stages, each its own tile and addend of y
    uint32_t k_len, base_tiles;
    size_t part_stride;
    uint32_t bn;         // activation rows per tile, at most (and rows of a box of the activation map)
    uint32_t stages;
    uint32_t T;
    LinGroups groups;
    uint32_t row_tiles[kMaxLinGroups];  // tiles of 128 weight rows per group
    uint32_t col_tiles;                 // tiles of bn activation rows per group
    const int32_t* moe_tiles;   // count, then (expert, first row) pairs; null: host groups
    const int32_t* moe_offsets;
    uint32_t moe_rows;          // weight rows per expert
    float* y;
    uint32_t y_stride;
    bf16* glu_out;
    uint32_t glu_stride;
    int glu_kind;
    float glu_limit;
    HeadSplit heads;
    uint32_t tmem_cols;
    unsigned int* err;
};

struct GemmTile {
    uint32_t w_row, w_left;  // first weight row, rows of the product left from there
    uint32_t x_row, n;       // first activation row, rows of the tile
    uint32_t y_row, y_col;
    uint32_t k0, n_k;        // stages
    size_t y_off;            // of the addend
};

__device__ __forceinline__ bool locate_tile(const GemmParams& p, uint32_t tile, GemmTile& t) {
    t.k0 = 0;
    t.n_k = p.n_k;
    t.y_off = 0;
    if (p.k_parts > 1) {
        const uint32_t part = tile / p.base_tiles;
        if (part >= p.k_parts) return false;
        tile -= part * p.base_tiles;
        t.k0 = part * p.k_len;
        t.n_k = p.n_k - t.k0 < p.k_len ? p.n_k - t.k0 : p.k_len;
        t.y_off = part * p.part_stride;
    }
    if (p.moe_tiles) {
        const uint32_t rt = p.row_tiles[0];
        const uint32_t ct = tile / rt, r = tile % rt;
        if (ct >= (uint32_t)p.moe_tiles[0]) return false;
        const uint32_t e = (uint32_t)p.moe_tiles[1 + 2 * ct], x0 = (uint32_t)p.moe_tiles[2 + 2 * ct];
        const uint32_t left = (uint32_t)p.moe_offsets[e + 1] - x0;
        t.w_row = e * p.moe_rows + r * 128;
        t.w_left = p.moe_rows - r * 128;
        t.x_row = x0;
        t.n = left < p.bn ? left : p.bn;
        t.y_row = x0;
        t.y_col = r * 128;
        return true;
    }
    for (uint32_t g = 0; g < p.groups.n; ++g) {
        const uint32_t rt = p.row_tiles[g], cnt = rt * p.col_tiles;
        if (tile < cnt) {
            const uint32_t ct = tile / rt, r = tile % rt;
            const LinGroup& G = p.groups.g[g];
            const uint32_t t0 = ct * p.bn;
            t.w_row = G.w_row + r * 128;
            t.w_left = G.rows - r * 128;
            t.x_row = G.x_row + t0;
            t.n = p.T - t0 < p.bn ? p.T - t0 : p.bn;
            t.y_row = t0;
            t.y_col = G.y_col + r * 128;
            return true;
        }
        tile -= cnt;
    }
    return false;
}

enum Epilogue { EPI_F32, EPI_GLU, EPI_HEADS };

template <int EPI>
__global__ void __launch_bounds__(GB_THREADS, 1)
gemm_bf16_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x,
                 const __grid_constant__ GemmParams p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ __align__(8) unsigned long long bars[2 * GB_MAX_STAGES + 4];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    pdl_launch_dependents();
    const uint32_t smem32 = ((uint32_t)__cvta_generic_to_shared(smem) + 1023u) & ~1023u;
    const uint32_t bar32 = (uint32_t)__cvta_generic_to_shared(bars);
    auto full = [&](uint32_t s) { return bar32 + s * 8; };
    auto empty = [&](uint32_t s) { return bar32 + (GB_MAX_STAGES + s) * 8; };
    auto acc_full = [&](uint32_t a) { return bar32 + (2 * GB_MAX_STAGES + a) * 8; };
    auto acc_empty = [&](uint32_t a) { return bar32 + (2 * GB_MAX_STAGES + 2 + a) * 8; };
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t stage_bytes = GB_A_BYTES + p.bn * 128;
    const uint32_t acc_cols = p.tmem_cols / 2;

    if (tid == 0) {
        for (uint32_t s = 0; s < p.stages; ++s) {
            mbar_init(full(s), 1);
            mbar_init(empty(s), 1);
        }
        for (uint32_t a = 0; a < 2; ++a) {
            mbar_init(acc_full(a), 1);
            mbar_init(acc_empty(a), GB_EPI_WARPS);
        }
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        const uint32_t slot = (uint32_t)__cvta_generic_to_shared(&tmem_slot);
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(slot), "r"(p.tmem_cols)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    volatile int* ab = &abort_flag;
    pdl_wait();

    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;  // stages issued so far
            bool alive = true;
            GemmTile t;
            for (uint32_t tile = blockIdx.x; alive && locate_tile(p, tile, t); tile += gridDim.x) {
                for (uint32_t k = 0; k < t.n_k; ++k, ++it) {
                    const uint32_t s = it % p.stages, round = it / p.stages;
                    if (round > 0) alive = mbar_wait(empty(s), (round - 1) & 1u, ab, p.err);
                    if (!alive) break;
                    const uint32_t a = smem32 + s * stage_bytes;
                    mbar_expect_tx(full(s), stage_bytes);
                    tensor_copy_2d(a, &map_w, (t.k0 + k) * 128, t.w_row, full(s));
                    tensor_copy_2d(a + GB_A_BYTES, &map_x, (t.k0 + k) * 128, t.x_row, full(s));
                    mbar_arrive(full(s));
                }
            }
            if (!alive) {  // copies still in flight land before the CTA may retire
                for (uint32_t back = 1; back <= p.stages && back <= it; ++back) {
                    const uint32_t j = it - back;
                    for (uint32_t i = 0; i < kSpinLimit; ++i)
                        if (mbar_try_wait(full(j % p.stages), (j / p.stages) & 1u)) break;
                }
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            uint32_t it = 0, n_tile = 0;
            bool alive = true;
            GemmTile t;
            for (uint32_t tile = blockIdx.x; alive && locate_tile(p, tile, t); tile += gridDim.x, ++n_tile) {
                const uint32_t a_id = n_tile & 1u, use = n_tile >> 1;
                if (use > 0) alive = mbar_wait(acc_empty(a_id), (use - 1) & 1u, ab, p.err);
                if (!alive) break;
                tc_fence_after();
                const uint32_t idesc = idesc_bf16(128, (t.n + 15u) & ~15u);
                const uint32_t d = tmem + a_id * acc_cols;
                for (uint32_t k = 0; k < t.n_k; ++k, ++it) {
                    const uint32_t s = it % p.stages;
                    alive = mbar_wait(full(s), (it / p.stages) & 1u, ab, p.err);
                    if (!alive) break;
                    tc_fence_after();
                    const uint32_t a = smem32 + s * stage_bytes;
                    const uint64_t ad = smem_desc_sw128(a), bd = smem_desc_sw128(a + GB_A_BYTES);
#pragma unroll
                    for (uint32_t k16 = 0; k16 < 4; ++k16)
                        tc_mma_f16(d, ad + 2 * k16, bd + 2 * k16, idesc, (k | k16) != 0 ? 1u : 0u);
                    tc_commit(empty(s));
                }
                if (alive) tc_commit(acc_full(a_id));
            }
            if (!alive) *ab = 1;
        }
        __syncwarp();
    } else {
        const uint32_t quarter = warp & 3u, half = (warp - 2) >> 2;
        uint32_t n_tile = 0;
        bool alive = true;
        GemmTile t;
        for (uint32_t tile = blockIdx.x; alive && locate_tile(p, tile, t); tile += gridDim.x, ++n_tile) {
            const uint32_t a_id = n_tile & 1u, use = n_tile >> 1;
            alive = mbar_wait(acc_full(a_id), use & 1u, ab, p.err);
            alive = __all_sync(0xFFFFFFFFu, alive);
            if (!alive) break;
            tc_fence_after();
            const uint32_t taddr = tmem + a_id * acc_cols + ((quarter * 32u) << 16);
            const uint32_t j = quarter * 32u + lane;
            bf16* split = nullptr;  // this lane's column of the two arrays
            uint32_t split_step = 0;
            if (EPI == EPI_HEADS && j < t.w_left) {
                const HeadSplit& H = p.heads;
                const uint32_t row = t.w_row + j, n0 = H.heads * H.d0, of = row < n0 ? row : row - n0;
                const uint32_t d = row < n0 ? H.d0 : H.d1, pitch = row < n0 ? H.pitch0 : H.pitch1;
                split_step = H.heads * pitch;
                split = (row < n0 ? H.out0 : H.out1) + (size_t)t.y_row * split_step + (of / d) * pitch + of % d;
            }
            for (uint32_t c = half * 32u; c < t.n; c += 64u) {
                uint32_t v[32];
                tc_ld32(taddr + c, v);
                tc_wait_ld();
                if (EPI == EPI_HEADS) {
                    if (split) {
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                            if (c + i < t.n) split[(size_t)(c + i) * split_step] = __float2bfloat16_rn(__uint_as_float(v[i]));
                    }
                } else if (EPI == EPI_GLU) {
                    const uint32_t up = lane >> 4;
                    const uint32_t f = ((t.y_col + quarter * 32u) >> 1) + (lane & 15u);
                    const bool ok = quarter * 32u < t.w_left;
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        const float lo = __uint_as_float(v[i]), hi = __uint_as_float(v[16 + i]);
                        const float got = __shfl_xor_sync(0xFFFFFFFFu, up ? lo : hi, 16);
                        const float g = up ? got : lo, u = up ? hi : got;
                        const uint32_t row = c + up * 16u + i;
                        if (ok && row < t.n)
                            p.glu_out[(size_t)(t.y_row + row) * p.glu_stride + f] =
                                __float2bfloat16_rn(glu_value(g, u, p.glu_kind, p.glu_limit));
                    }
                } else if (j < t.w_left) {
                    float* o = p.y + t.y_off + (size_t)(t.y_row + c) * p.y_stride + t.y_col + j;
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (c + i < t.n) o[(size_t)i * p.y_stride] = __uint_as_float(v[i]);
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(acc_empty(a_id));
        }
    }

    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        // Abandoned: the instructions in flight get a bounded chance to finish. The phase of the commit is not known
        // here, so a barrier that nothing else uses any more tells: it is initialised anew.
        if (abort_flag && lane == 0) {
            mbar_init(acc_empty(0), 1);
            tc_commit(acc_empty(0));
            for (uint32_t i = 0; i < kSpinLimit; ++i)
                if (mbar_try_wait(acc_empty(0), 0)) break;
        }
        __syncwarp();
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(p.tmem_cols) : "memory");
    }
}

// Tile height (activation rows) and number of K runs: the cheapest by a count of cycles. A 64-K stage costs four
// instructions of about 128 cycles whatever N is, or the time its copies take at about 80 bytes a cycle and SM; the last
// tile's drain comes on top, and writing and reading the addends at about 2600 bytes a cycle.
struct Plan {
    uint32_t bn, parts;
};
Plan plan_tiles(uint32_t row_tiles, uint32_t T, uint32_t n_k, uint32_t max_parts, size_t out_floats, uint32_t sms) {
    Plan best{32, 1};
    uint64_t best_cost = ~0ull;
    for (uint32_t parts = 1; parts <= max_parts; parts <<= 1) {
        if (parts > 1 && n_k / parts < 8) break;
        for (uint32_t bn = 32; bn <= 256; bn <<= 1) {
            if (bn > 32 && bn / 2 >= T) break;  // half the height holds all rows
            const uint64_t tiles = (uint64_t)row_tiles * ((T + bn - 1) / bn) * parts, waves = (tiles + sms - 1) / sms;
            const uint32_t copy = (128 + bn) * 128 / 80, k = (n_k + parts - 1) / parts;
            const uint64_t cost = waves * k * (copy > 512 ? copy : 512) + bn * 34ull + (parts > 1 ? out_floats * parts * 8 / 2600 : 0);
            if (cost < best_cost) {
                best_cost = cost;
                best = Plan{bn, parts};
            }
        }
    }
    return best;
}

int launch(const DenseWeight& W, const bf16* x, uint32_t x_pitch, uint32_t x_rows, GemmParams& p, uint64_t tiles,
           Epilogue epi, cudaStream_t st) {
    const uint32_t stage_bytes = GB_A_BYTES + p.bn * 128;
    p.n_k = W.kp / 64;
    if (p.k_parts > 1) {
        p.k_len = (p.n_k + p.k_parts - 1) / p.k_parts;
        p.k_parts = (p.n_k + p.k_len - 1) / p.k_len;  // no empty run
        p.base_tiles = (uint32_t)tiles;
        tiles *= p.k_parts;
    }
    p.stages = GB_SMEM / stage_bytes;
    if (p.stages > GB_MAX_STAGES) p.stages = GB_MAX_STAGES;
    p.tmem_cols = 2 * p.bn;
    int rc = device_error_word(&p.err);
    if (rc != ZQ_OK) return rc;
    CUtensorMap mw, mx;
    if ((rc = tensor_map_2d(W.w, (uint64_t)W.kp * 2, W.rows, 128, 128, 128, &mw)) != ZQ_OK) return rc;
    if ((rc = tensor_map_2d(x, (uint64_t)x_pitch * 2, x_rows, 128, p.bn, 128, &mx)) != ZQ_OK) return rc;
    auto kern = epi == EPI_GLU ? gemm_bf16_kernel<EPI_GLU> : epi == EPI_HEADS ? gemm_bf16_kernel<EPI_HEADS> : gemm_bf16_kernel<EPI_F32>;
    const uint32_t smem = p.stages * stage_bytes + 1024;
    ZQ_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - 1024));
    const uint32_t grid = tiles < (uint64_t)sm_count() ? (uint32_t)tiles : (uint32_t)sm_count();
    const cudaError_t e = launch_pdl(kern, dim3(grid), dim3(GB_THREADS), smem, st, mw, mx, p);
    if (e != cudaSuccess) return cuda_fail(e);
    return ZQ_OK;
}

}  // namespace

int launch_gemm_bf16(const DenseWeight& W, const LinGroups& G, const bf16* x, uint32_t x_rows, uint32_t T, float* y,
                     uint32_t y_stride, bf16* glu_out, uint32_t glu_stride, const GluSpec* glu, cudaStream_t st,
                     Addends* add, size_t y_floats) {
    if (add) *add = Addends{};
    if (T == 0) return ZQ_OK;
    if (G.n == 0 || G.n > kMaxLinGroups) return ZQ_ERR_BAD_ARG;
    GemmParams p{};
    p.T = T;
    p.groups = G;
    uint32_t rt = 0;
    for (uint32_t g = 0; g < G.n; ++g) {
        p.row_tiles[g] = (G.g[g].rows + 127) / 128;
        rt += p.row_tiles[g];
    }
    const size_t out_floats = (size_t)T * y_stride;
    const uint32_t max_parts = add && !glu && G.n == 1 && out_floats ? (uint32_t)(y_floats / out_floats < 8 ? y_floats / out_floats : 8) : 1;
    const Plan plan = plan_tiles(rt, T, W.kp / 64, max_parts ? max_parts : 1, out_floats, (uint32_t)sm_count());
    p.bn = plan.bn;
    p.k_parts = plan.parts;
    p.part_stride = out_floats;
    p.col_tiles = (T + p.bn - 1) / p.bn;
    p.y = y;
    p.y_stride = y_stride;
    p.glu_out = glu_out;
    p.glu_stride = glu_stride;
    if (glu) {
        p.glu_kind = glu->kind;
        p.glu_limit = glu->limit;
    }
    const int rc = launch(W, x, W.kp, x_rows, p, (uint64_t)rt * p.col_tiles, glu ? EPI_GLU : EPI_F32, st);
    if (add && p.k_parts > 1) *add = Addends{p.k_parts, out_floats};
    return rc;
}

int launch_gemm_bf16_heads(const DenseWeight& W, const bf16* x, uint32_t x_pitch, uint32_t x_rows, uint32_t T,
                           const HeadSplit& split, cudaStream_t st) {
    if (T == 0) return ZQ_OK;
    if (W.rows != split.heads * (split.d0 + split.d1)) return ZQ_ERR_BAD_ARG;
    GemmParams p{};
    p.T = T;
    p.groups = one_group(W.rows);
    p.row_tiles[0] = (W.rows + 127) / 128;
    p.bn = plan_tiles(p.row_tiles[0], T, W.kp / 64, 1, 0, (uint32_t)sm_count()).bn;
    p.k_parts = 1;
    p.col_tiles = (T + p.bn - 1) / p.bn;
    p.heads = split;
    return launch(W, x, x_pitch, x_rows, p, (uint64_t)p.row_tiles[0] * p.col_tiles, EPI_HEADS, st);
}

int launch_moe_grouped(const MoeWeights& M, const MoeRouting& R, const bf16* xs, uint32_t T, uint32_t bn, bf16* hidden,
                       float* parts, cudaStream_t st) {
    if (T == 0) return ZQ_OK;
    const uint32_t pairs = T * M.top;
    // at most one partly filled tile per expert beside the full ones
    const uint64_t col_tiles = (uint64_t)pairs / bn + M.experts;
    GemmParams p{};
    p.k_parts = 1;
    p.bn = bn;
    p.moe_tiles = R.tiles;
    p.moe_offsets = R.offsets;
    p.moe_rows = 2 * M.ffp;
    p.row_tiles[0] = (p.moe_rows + 127) / 128;
    p.glu_out = hidden;
    p.glu_stride = M.ffp;
    p.glu_kind = M.glu.kind;
    p.glu_limit = M.glu.limit;
    int rc = launch(M.gate_up, xs, M.gate_up.kp, pairs, p, col_tiles * p.row_tiles[0], EPI_GLU, st);
    if (rc != ZQ_OK) return rc;
    p.moe_rows = M.width;
    p.row_tiles[0] = (p.moe_rows + 127) / 128;
    p.glu_out = nullptr;
    p.y = parts;
    p.y_stride = M.width;
    return launch(M.down, hidden, M.down.kp, pairs, p, col_tiles * p.row_tiles[0], EPI_F32, st);
}

}  // namespace zq
