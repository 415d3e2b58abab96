// C entry points of the single mechanisms (include/zq.h): argument checks around the launchers of dense.h.
#include <string.h>

#include <new>
#include <vector>

#include "dense.h"

struct zq_dense {
    zq::DenseWeight w;
    bool glu = false;
};

using namespace zq;

namespace {

bool known(int precision) { return precision == ZQ_PRECISION_BF16 || precision == ZQ_PRECISION_F32; }
bool is_f32(int precision) { return precision == ZQ_PRECISION_F32; }

GqaShape shape_of(const zq_gqa* g) {
    return GqaShape{g->heads, g->kv_heads, g->dim, g->vdim, pad_to(g->dim, 16), pad_to(g->vdim, 16), g->ctx, g->slots};
}
bool valid(const zq_gqa* g) {
    return g && g->heads && g->kv_heads && g->heads % g->kv_heads == 0 && g->dim && g->vdim && g->ctx && g->slots;
}

bool valid(const zq_memory_shape* s) {
    return s && s->heads && s->dim && s->vdim && s->gate_cap > 0.0f && s->ld >= 2 * s->heads * (s->dim + s->vdim + 1);
}
bool valid(const zq_delta_shape* s) {
    return s && s->heads && s->kv_heads && s->heads % s->kv_heads == 0 && s->dim && s->vdim && s->taps && s->a_rank && s->g_rank &&
           s->ld >= 2 * s->kv_heads * s->dim + s->heads * (s->vdim + 1) + s->a_rank + s->g_rank;
}
DeltaArgs args_of(const zq_delta_shape* s) {
    DeltaArgs a{};
    a.heads = s->heads;
    a.kv_heads = s->kv_heads;
    a.dim = s->dim;
    a.vdim = s->vdim;
    a.taps = s->taps;
    a.a_rank = s->a_rank;
    a.g_rank = s->g_rank;
    a.ld = s->ld;
    a.eps = s->eps;
    a.low.k = s->a_rank > s->g_rank ? s->a_rank : s->g_rank;
    a.low.kp = pad64(a.low.k);
    return a;
}
bool valid(const zq_latent_shape* s) {
    return s && s->heads && s->dim && s->vdim && s->rank && s->rot % 2 == 0 && s->ctx && s->slots && s->ld >= s->heads * (s->dim + s->rot);
}
LatentShape shape_of(const zq_latent_shape* s) {
    return LatentShape{s->heads, s->dim, s->rot, s->vdim, s->rank, pad_to(s->rank + s->rot, 16), s->ctx, s->slots};
}

int upload(const zq_bf16_ref* a, const zq_bf16_ref* b, zq_stream stream, zq_dense** out) {
    if (!a || !a->data || !a->rows || !a->cols || !out) return ZQ_ERR_BAD_ARG;
    if (b && (!b->data || b->rows != a->rows || b->cols != a->cols)) return ZQ_ERR_BAD_ARG;
    *out = nullptr;
    zq_dense* d = new (std::nothrow) zq_dense;
    if (!d) return ZQ_ERR_NO_MEM;
    d->glu = b != nullptr;
    d->w.k = a->cols;
    d->w.kp = pad64(a->cols);
    d->w.rows = b ? 2 * pad64(a->rows) : a->rows;
    const size_t n = (size_t)d->w.rows * d->w.kp;
    std::vector<uint16_t> host;
    try {
        host.assign(n, 0);
    } catch (...) {
        delete d;
        return ZQ_ERR_NO_MEM;
    }
    for (uint32_t r = 0; r < a->rows; ++r) {
        memcpy(host.data() + (size_t)(b ? glu_row(r, false) : r) * d->w.kp, a->data + (size_t)r * a->cols, (size_t)a->cols * 2);
        if (b) memcpy(host.data() + (size_t)glu_row(r, true) * d->w.kp, b->data + (size_t)r * b->cols, (size_t)b->cols * 2);
    }
    cudaError_t e = cudaMalloc(reinterpret_cast<void**>(&d->w.w), n * 2);
    if (e == cudaSuccess) e = cudaMemcpyAsync(d->w.w, host.data(), n * 2, cudaMemcpyHostToDevice, as_stream(stream));
    if (e == cudaSuccess) e = cudaStreamSynchronize(as_stream(stream));
    if (e != cudaSuccess) {
        cudaFree(d->w.w);
        delete d;
        return cuda_fail(e);
    }
    *out = d;
    return ZQ_OK;
}

}  // namespace

extern "C" {

int zq_dense_upload(const zq_bf16_ref* w, zq_stream stream, zq_dense** out) { return upload(w, nullptr, stream, out); }

int zq_dense_upload_glu(const zq_bf16_ref* gate, const zq_bf16_ref* up, zq_stream stream, zq_dense** out) {
    return up ? upload(gate, up, stream, out) : ZQ_ERR_BAD_ARG;
}

int zq_dense_free(zq_dense* w) {
    if (w) cudaFree(w->w.w);
    delete w;
    return ZQ_OK;
}

uint32_t zq_dense_pitch(uint32_t k) { return pad64(k); }

int zq_dense_linear(const zq_dense* w, const void* d_x, uint32_t rows, float* d_y, int precision, zq_stream stream) {
    if (!w || w->glu || !d_x || !d_y || !known(precision)) return ZQ_ERR_BAD_ARG;
    return launch_dense_linear(w->w, one_group(w->w.rows), d_x, rows, rows, d_y, w->w.rows, is_f32(precision), as_stream(stream));
}

int zq_dense_glu(const zq_dense* w, const void* d_x, uint32_t rows, void* d_out, int kind, float limit, int precision,
                 zq_stream stream) {
    if (!w || !w->glu || !d_x || !d_out || !known(precision) || (kind != ZQ_GLU_SILU && kind != ZQ_GLU_CLAMPED))
        return ZQ_ERR_BAD_ARG;
    GluSpec g;
    g.kind = kind == ZQ_GLU_SILU ? GLU_SILU : GLU_CLAMPED;
    g.limit = limit;
    return launch_dense_glu(w->w, d_x, rows, d_out, g, is_f32(precision), as_stream(stream));
}

int zq_gqa_cache_write(const zq_gqa* g, const float* d_qkv, const float* d_q_norm, const float* d_k_norm,
                       const float* d_vmix, float* d_v_first, void* d_q, void* d_k_cache, void* d_v_cache,
                       const int32_t* d_pos, const int32_t* d_slots, uint32_t rows, int precision, zq_stream stream) {
    if (!valid(g) || !d_qkv || !d_q_norm || !d_k_norm || (d_vmix && !d_v_first) || !d_q || !d_k_cache || !d_v_cache ||
        !d_pos || !d_slots || !known(precision))
        return ZQ_ERR_BAD_ARG;
    QkvPostArgs a{};
    a.s = shape_of(g);
    a.qkv = d_qkv;
    a.q_norm = d_q_norm;
    a.k_norm = d_k_norm;
    a.eps = g->norm_eps;
    a.temp_coef = g->temp_coef;
    a.temp_every = g->temp_every;
    a.vmix = d_vmix;
    a.v_first = d_v_first;
    a.q = d_q;
    a.kc = d_k_cache;
    a.vc = d_v_cache;
    a.pos = d_pos;
    a.slots = d_slots;
    return launch_qkv_post(a, rows, is_f32(precision), as_stream(stream));
}

size_t zq_gqa_work_bytes(const zq_gqa* g, uint32_t rows) { return valid(g) ? gqa_work_bytes(shape_of(g), rows) : 0; }

int zq_gqa_attention(const zq_gqa* g, const void* d_q, const void* d_k_cache, const void* d_v_cache, void* d_out,
                     const int32_t* d_pos, const int32_t* d_slots, uint32_t rows, int one_sequence, uint32_t pos0,
                     void* d_work, int precision, zq_stream stream) {
    if (!valid(g) || !d_q || !d_k_cache || !d_v_cache || !d_out || !d_pos || !d_slots || !d_work || !known(precision))
        return ZQ_ERR_BAD_ARG;
    return launch_gqa_attention(shape_of(g), d_q, d_k_cache, d_v_cache, d_out, pad64(g->heads * g->vdim), g->scale, d_pos,
                                d_slots, rows, one_sequence != 0, pos0, d_work, is_f32(precision), as_stream(stream));
}

int zq_token_shift(const float* d_h, const float* d_mu, const float* d_prev, const int32_t* d_slots, uint32_t n_mix,
                   uint32_t rows, uint32_t width, void* d_mix, int precision, zq_stream stream) {
    if (!d_h || !d_mu || !d_prev || !d_slots || !d_mix || !n_mix || !width || !known(precision)) return ZQ_ERR_BAD_ARG;
    return launch_token_shift(d_h, d_mu, d_prev, d_slots, n_mix, rows, rows, width, d_mix, is_f32(precision), as_stream(stream));
}

size_t zq_wkv_work_floats(uint32_t heads, uint32_t dim, uint32_t rows) {
    return (size_t)rows * heads * dim + wkv_chunk_floats(heads, dim, rows);
}

int zq_wkv(const float* d_in, uint32_t heads, uint32_t dim, uint32_t rank, const zq_dense* w2, const float* d_w0,
           const float* d_u, const float* d_norm, float eps, float* d_state, const int32_t* d_slots, uint32_t rows,
           int one_sequence, float* d_work, void* d_out, int precision, zq_stream stream) {
    if (!d_in || !heads || !dim || !rank || !w2 || w2->glu || w2->w.rows != heads * dim || w2->w.k != rank || !d_w0 || !d_u ||
        !d_norm || !d_state || !d_slots || !d_work || !d_out || !known(precision))
        return ZQ_ERR_BAD_ARG;
    WkvArgs a{};
    a.heads = heads;
    a.dim = dim;
    a.rank = rank;
    a.rank_p = w2->w.kp;
    a.ld = 4 * heads * dim + rank;
    a.rkvg = d_in;
    a.w2 = w2->w.w;
    a.w0 = d_w0;
    a.u = d_u;
    a.norm = d_norm;
    a.eps = eps;
    a.state = d_state;
    a.slots = d_slots;
    a.out = d_out;
    a.out_pitch = pad64(heads * dim);
    a.decay = d_work;
    a.chunk = d_work + (size_t)rows * heads * dim;
    return launch_wkv(a, rows, one_sequence != 0, is_f32(precision), as_stream(stream));
}

size_t zq_memory_work_floats(const zq_memory_shape* s, uint32_t rows) {
    return valid(s) ? memory_work_floats(s->heads, s->dim, s->vdim, rows) : 0;
}

int zq_memory(const zq_memory_shape* s, const float* d_in, const float* d_i_bias, const float* d_f_bias, const float* d_norm,
              float* d_S, float* d_n, float* d_m, const int32_t* d_slots, uint32_t rows, int one_sequence, float* d_work,
              void* d_out, int precision, zq_stream stream) {
    if (!valid(s) || !d_in || !d_i_bias || !d_f_bias || !d_norm || !d_S || !d_n || !d_m || !d_slots || !d_work || !d_out ||
        !known(precision))
        return ZQ_ERR_BAD_ARG;
    MemoryArgs a{};
    a.heads = s->heads;
    a.dim = s->dim;
    a.vdim = s->vdim;
    a.ld = s->ld;
    a.in = d_in;
    a.i_bias = d_i_bias;
    a.f_bias = d_f_bias;
    a.gate_cap = s->gate_cap;
    a.norm = d_norm;
    a.eps = s->eps;
    a.S = d_S;
    a.n = d_n;
    a.m = d_m;
    a.slots = d_slots;
    a.out = d_out;
    a.out_pitch = pad64(s->heads * s->vdim);
    a.work = d_work;
    return launch_memory(a, rows, one_sequence != 0, is_f32(precision), as_stream(stream));
}

size_t zq_delta_work_floats(const zq_delta_shape* s, uint32_t rows) { return valid(s) ? delta_work_floats(args_of(s), rows) : 0; }

int zq_delta(const zq_delta_shape* s, const float* d_in, const float* d_conv, const float* d_A_log, const float* d_dt_bias,
             const zq_dense* low, const float* d_norm, float* d_S, float* d_ring, const int32_t* d_pos, const int32_t* d_slots,
             uint32_t rows, int one_sequence, float* d_work, void* d_out, int precision, zq_stream stream) {
    if (!valid(s) || !d_in || !d_conv || !d_A_log || !d_dt_bias || !low || low->glu || !d_norm || !d_S || (s->taps > 1 && !d_ring) ||
        !d_pos || !d_slots || !d_work || !d_out || !known(precision))
        return ZQ_ERR_BAD_ARG;
    DeltaArgs a = args_of(s);
    if (low->w.rows != s->heads * (s->dim + s->vdim) || low->w.k != a.low.k) return ZQ_ERR_BAD_ARG;
    a.in = d_in;
    a.conv = d_conv;
    a.A_log = d_A_log;
    a.dt_bias = d_dt_bias;
    a.low = low->w;
    a.norm = d_norm;
    a.S = d_S;
    a.ring = d_ring;
    a.pos = d_pos;
    a.slots = d_slots;
    a.out = d_out;
    a.out_pitch = pad64(s->heads * s->vdim);
    a.work = d_work;
    a.max_rows = rows;
    return launch_delta(a, rows, one_sequence != 0, is_f32(precision), as_stream(stream));
}

size_t zq_latent_work_bytes(const zq_latent_shape* s, uint32_t rows, int precision) {
    return valid(s) ? latent_work_bytes(shape_of(s), rows, is_f32(precision)) : 0;
}

int zq_latent_attention(const zq_latent_shape* s, const float* d_in, const float* d_norm, const float* d_freq,
                        const zq_dense* up, void* d_cache, const int32_t* d_pos, const int32_t* d_slots, uint32_t rows,
                        int one_sequence, uint32_t slot0, uint32_t pos0, void* d_work, void* d_out, int precision,
                        zq_stream stream) {
    if (!valid(s) || !d_in || (s->rot && !d_freq) || !up || up->glu || up->w.rows != s->heads * (s->dim + s->vdim) ||
        up->w.k != s->rank || !d_cache || !d_pos || !d_slots || !d_work || !d_out || !known(precision) ||
        (one_sequence && (slot0 >= s->slots || pos0 >= s->ctx || rows > s->ctx - pos0)))
        return ZQ_ERR_BAD_ARG;
    LatentArgs a{};
    a.s = shape_of(s);
    a.in = d_in;
    a.ld = s->ld;
    a.own = d_norm != nullptr;
    a.norm = d_norm;
    a.eps = s->eps;
    a.scale = s->scale;
    a.freq = d_freq;
    a.up = up->w;
    a.cache = d_cache;
    a.pos = d_pos;
    a.slots = d_slots;
    a.slot0 = slot0;
    a.out = d_out;
    a.out_pitch = pad64(s->heads * s->vdim);
    a.work = d_work;
    a.max_rows = rows;
    return launch_latent(a, rows, one_sequence != 0, pos0, is_f32(precision), as_stream(stream));
}

int zq_route(const float* d_logits, uint32_t stride, uint32_t experts, uint32_t top, const float* d_bias, int kind,
             int32_t* d_ids, float* d_weights, uint32_t rows, zq_stream stream) {
    if (!d_logits || !d_ids || !d_weights || !experts || !top || top > experts || stride < experts ||
        (kind != ZQ_ROUTE_SIGMOID && kind != ZQ_ROUTE_SOFTMAX))
        return ZQ_ERR_BAD_ARG;
    MoeRouting R{};
    R.ids = d_ids;
    R.weights = d_weights;
    return launch_route(d_logits, stride, experts, top, d_bias, kind == ZQ_ROUTE_SOFTMAX ? ROUTE_SOFTMAX : ROUTE_SIGMOID, R, rows,
                        as_stream(stream));
}

}  // extern "C"
