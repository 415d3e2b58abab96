// Device-resident engine for decoders over bf16 weights whose layers mix tokens by attention or by a recurrence. Like the
// other engines (engine.cu) it uploads every tensor once, allocates cache, states and scratch once, and runs a forward
// pass as a fixed sequence of launches on the caller's stream; a decode step is recorded once and replayed.
//
// One forward pass covers either T consecutive tokens of one sequence (prefill, in pieces of up to max_rows) or one
// token of each of several sequences (decode). Rows find their position and slot in device memory.
// Launches of a decode step: [embedding + norm (+ token shift)] | qkv | q/k norm, temperature, value mixing, cache
// write and attention per key range | ranges | o | norm + residual + norm | gate, up and their unit | down | norm +
// residual + next norm (+ token shift); a recurrent layer: r, k, v, g, w1 in one launch | decay, recurrence, head norm
// and gate | o | ...; experts: router | routing | the chosen and the shared experts' units | their downs. A layer whose
// sublayers read the same norm has the router's rows in its mixer's first product, and one sum for both at its end; for a
// few rows the feed-forward's products, which are bound by memory, run beside the mixer's small kernels on a second stream.
#include <math.h>

#include <algorithm>
#include <new>

#include "dense.h"
#include "engine_common.h"

namespace zq {
namespace {

__global__ void set_row_kernel(int32_t* tokens, int32_t* pos, int32_t* slots, uint32_t* rec, uint32_t token, uint32_t p,
                               uint32_t slot) {
    tokens[0] = (int32_t)token;
    pos[0] = (int32_t)p;
    slots[0] = (int32_t)slot;
    *rec = 0;
}
__global__ void set_rows_kernel(int32_t* pos, int32_t* slots, uint32_t pos0, uint32_t slot, uint32_t n) {
    const uint32_t i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    pos[i] = (int32_t)(pos0 + i);
    slots[i] = (int32_t)slot;
}
__global__ void feed_row_kernel(int32_t* tokens, int32_t* pos, uint32_t* rec, const int32_t* arg, uint32_t* record) {
    const uint32_t t = (uint32_t)*arg;
    record[*rec] = t;
    tokens[0] = (int32_t)t;
    pos[0] += 1;
    *rec += 1;
}

struct AttentionLayer {
    DenseWeight qkv, o;
    float *q_norm = nullptr, *k_norm = nullptr, *vmix = nullptr;
    GqaShape s{};
    float scale = 0, temp_coef = 0, temp_every = 0;
    bool v_mix = false, v_first = false;
    void *kc = nullptr, *vc = nullptr;
};
struct WkvLayer {
    DenseWeight in, w2, o;  // in: r | k | v | g | w1 rows
    float *mu = nullptr, *w0 = nullptr, *u = nullptr, *norm = nullptr;
    uint32_t heads = 0, dim = 0, rank = 0;
    float *state = nullptr, *prev = nullptr;
};
struct MemoryLayer {
    DenseWeight in, o;  // in: q | k | v | gate | i | f (| router) rows
    float *i_bias = nullptr, *f_bias = nullptr, *norm = nullptr;
    float gate_cap = 0;
    uint32_t heads = 0, dim = 0, vdim = 0;
    float *S = nullptr, *n = nullptr, *m = nullptr;
};
struct DeltaLayer {
    DenseWeight in, o;  // in: q | k | v | beta | a1 | g1 (| router) rows
    DeltaArgs args{};   // without the pointers of a pass
};
struct LatentLayer {
    DenseWeight in, o, up;  // in: q (| dkv) (| router) rows; up: uk | uv rows
    LatentShape s{};
    float *norm = nullptr, *freq = nullptr;
    float scale = 0;
    bool own = true;
    void* cache = nullptr;
};
struct Layer {
    uint32_t mixer = 0, mlp = 0;
    bool parallel = false;    // x += mixer(n1(x)) + ff(n1(x))
    int32_t router_col = -1;  // column of the router logits in the mixer's first product; -1: a product of its own
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
    AttentionLayer att;
    WkvLayer wkv;
    MemoryLayer mem;
    DeltaLayer delta;
    LatentLayer lat;
    DenseWeight gate_up, down;
    GluSpec glu;
    MoeWeights moe;
    DenseWeight router;  // [experts (+ 1: the shared expert's gate)] rows
    float* router_bias = nullptr;
    int route_kind = ROUTE_SIGMOID;
    bool shared_gated = false;
};
// Part of a sequence's state that starts at zero: `bytes` per slot.
struct SlotState {
    char* base;
    size_t bytes;
};

}  // namespace
}  // namespace zq

using namespace zq;

struct zq_decoder {
    zq_decoder_config c{};
    bool f32 = false;
    DeviceArena arena;
    StepGraphs graphs;
    DenseWeight embed, head;
    float *embed_norm = nullptr, *final_norm = nullptr;
    std::vector<Layer> layers;
    std::vector<SlotState> states;
    uint32_t hp = 0, max_rows = 1;
    // activations
    float *x = nullptr, *y = nullptr, *h32 = nullptr, *proj = nullptr, *v_first = nullptr, *z = nullptr;
    float* y2 = nullptr;  // the feed-forward's product in a layer with parallel sublayers
    size_t y_floats = 0;
    Addends y_add;        // of the product that y holds
    void *h = nullptr, *mix = nullptr, *q = nullptr, *att = nullptr, *hid = nullptr;
    float *parts = nullptr, *decay = nullptr, *chunk = nullptr;
    bf16* xs = nullptr;
    void* work = nullptr;  // of the mixer that runs
    MoeRouting route{};
    float* logits = nullptr;  // [n_seq][vocab]
    int32_t *d_tokens = nullptr, *d_pos = nullptr, *d_slots = nullptr, *d_want = nullptr, *d_arg = nullptr;
    uint32_t *d_rec = nullptr, *d_record = nullptr;
    std::vector<uint32_t> seq_lens;
    float* trail = nullptr;
    uint32_t trail_rows = 0;
    // the feed-forward part beside a mixer
    cudaStream_t side = nullptr;
    cudaEvent_t forked = nullptr, joined = nullptr;
    ~zq_decoder() {
        if (forked) cudaEventDestroy(forked);
        if (joined) cudaEventDestroy(joined);
        if (side) cudaStreamDestroy(side);
    }
};

namespace {

// ------------------------------------------------------------------------------------------------ loading
struct Loader {
    zq_decoder* m;
    cudaStream_t st;
    std::vector<uint16_t> host;

    int put(DenseWeight* W, uint32_t rows, uint32_t k) {
        W->rows = rows;
        W->k = k;
        W->kp = pad64(k);
        host.assign((size_t)rows * W->kp, 0);
        return ZQ_OK;
    }
    int rows_from(const DenseWeight& W, const zq_bf16_ref& t, uint32_t rows, uint32_t at) {
        if (!rows) return ZQ_OK;
        if (!t.data || t.rows != rows || t.cols != W.k) return ZQ_ERR_BAD_ARG;
        for (uint32_t r = 0; r < rows; ++r)
            memcpy(host.data() + (size_t)(at + r) * W.kp, t.data + (size_t)r * W.k, (size_t)W.k * 2);
        return ZQ_OK;
    }
    // rows of t as they are, in a matrix that may have more columns
    int rows_cut(const DenseWeight& W, const zq_bf16_ref& t, uint32_t at) {
        if (!t.data || t.cols > W.k) return ZQ_ERR_BAD_ARG;
        for (uint32_t r = 0; r < t.rows; ++r)
            memcpy(host.data() + (size_t)(at + r) * W.kp, t.data + (size_t)r * t.cols, (size_t)t.cols * 2);
        return ZQ_OK;
    }
    int glu_from(const DenseWeight& W, const zq_bf16_ref& t, uint32_t rows, uint32_t at, bool up) {
        if (!t.data || t.rows != rows || t.cols != W.k) return ZQ_ERR_BAD_ARG;
        for (uint32_t r = 0; r < rows; ++r)
            memcpy(host.data() + (size_t)(at + glu_row(r, up)) * W.kp, t.data + (size_t)r * W.k, (size_t)W.k * 2);
        return ZQ_OK;
    }
    int send(DenseWeight* W) {
        int rc = m->arena.alloc_n(&W->w, host.size());
        if (rc != ZQ_OK) return rc;
        ZQ_CUDA(cudaMemcpyAsync(W->w, host.data(), host.size() * 2, cudaMemcpyHostToDevice, st));
        ZQ_CUDA(cudaStreamSynchronize(st));  // `host` is used again
        return ZQ_OK;
    }
    int matrix(DenseWeight* W, const zq_bf16_ref& t, uint32_t rows, uint32_t k) {
        int rc;
        if ((rc = put(W, rows, k)) || (rc = rows_from(*W, t, rows, 0))) return rc;
        return send(W);
    }
    int glu(DenseWeight* W, const zq_bf16_ref& gate, const zq_bf16_ref& up, uint32_t ff, uint32_t k) {
        int rc;
        if ((rc = put(W, 2 * pad64(ff), k)) || (rc = glu_from(*W, gate, ff, 0, false)) || (rc = glu_from(*W, up, ff, 0, true)))
            return rc;
        return send(W);
    }
    int vec(float** out, const float* v, size_t n) { return m->arena.upload_f32(out, v, n, st); }
};

#define RUN(expr)                                  \
    do {                                           \
        const int rc__ = (expr);                   \
        if (rc__ != ZQ_OK) return rc__;            \
    } while (0)

int zeroed(zq_decoder* m, void** out, size_t bytes, cudaStream_t st) {
    RUN(m->arena.alloc(out, bytes));
    ZQ_CUDA(cudaMemsetAsync(*out, 0, bytes, st));
    return ZQ_OK;
}

// A part of every sequence's state, zero at its start.
template <typename T>
int slot_state(zq_decoder* m, T** out, size_t per_slot, cudaStream_t st) {
    RUN(zeroed(m, reinterpret_cast<void**>(out), m->c.n_seq * per_slot * sizeof(T), st));
    m->states.push_back(SlotState{reinterpret_cast<char*>(*out), per_slot * sizeof(T)});
    return ZQ_OK;
}

// Rows of the router that a mixer's first product carries.
uint32_t router_rows(const zq_decoder_layer& s) {
    return s.parallel && s.mlp == ZQ_MLP_MOE ? s.experts + (s.shared_sg.data ? 1 : 0) : 0;
}
int put_router(Loader& L, const DenseWeight& W, const zq_decoder_layer& s, uint32_t at) {
    RUN(L.rows_from(W, s.router, s.experts, at));
    return s.shared_sg.data ? L.rows_from(W, s.shared_sg, 1, at + s.experts) : ZQ_OK;
}
// Matrices of the same width below one another, then the router's rows.
struct Part {
    const zq_bf16_ref* ref;
    uint32_t rows;
};
int stack(Loader& L, Layer& d, const zq_decoder_layer& s, DenseWeight* W, std::initializer_list<Part> parts) {
    uint32_t at = 0;
    for (const Part& p : parts) at += p.rows;
    RUN(L.put(W, at + router_rows(s), L.m->c.width));
    if (router_rows(s)) {
        d.router_col = (int32_t)at;
        RUN(put_router(L, *W, s, at));
    }
    at = 0;
    for (const Part& p : parts) {
        RUN(L.rows_from(*W, *p.ref, p.rows, at));
        at += p.rows;
    }
    return L.send(W);
}

int load_memory(zq_decoder* m, Loader& L, Layer& d, const zq_decoder_layer& s) {
    if (!s.heads || !s.dim || !s.vdim || !(s.gate_cap > 0.0f)) return ZQ_ERR_BAD_ARG;
    MemoryLayer& w = d.mem;
    const uint32_t H = s.heads, kd = H * s.dim, vd = H * s.vdim;
    w.heads = H;
    w.dim = s.dim;
    w.vdim = s.vdim;
    w.gate_cap = s.gate_cap;
    RUN(stack(L, d, s, &w.in, {{&s.q, kd}, {&s.k, kd}, {&s.v, vd}, {&s.g, vd}, {&s.i, H}, {&s.f, H}}));
    RUN(L.matrix(&w.o, s.o, m->c.width, vd));
    RUN(L.vec(&w.i_bias, s.i_bias, H));
    RUN(L.vec(&w.f_bias, s.f_bias, H));
    RUN(L.vec(&w.norm, s.mix_norm, vd));
    RUN(slot_state(m, &w.S, (size_t)kd * s.vdim, L.st));
    RUN(slot_state(m, &w.n, kd, L.st));
    return slot_state(m, &w.m, H, L.st);
}

int load_delta(zq_decoder* m, Loader& L, Layer& d, const zq_decoder_layer& s) {
    if (!s.heads || !s.kv_heads || s.heads % s.kv_heads || !s.dim || !s.vdim || !s.taps || !s.a1.rows || !s.g1.rows)
        return ZQ_ERR_BAD_ARG;
    DeltaLayer& w = d.delta;
    const uint32_t H = s.heads, kd = s.kv_heads * s.dim, hd = H * s.dim, vd = H * s.vdim, ch = 2 * kd + vd;
    const uint32_t rank = std::max(s.a1.rows, s.g1.rows);
    RUN(stack(L, d, s, &w.in, {{&s.q, kd}, {&s.k, kd}, {&s.v, vd}, {&s.b, H}, {&s.a1, s.a1.rows}, {&s.g1, s.g1.rows}}));
    RUN(L.matrix(&w.o, s.o, m->c.width, vd));
    DeltaArgs& a = w.args;
    a.heads = H;
    a.kv_heads = s.kv_heads;
    a.dim = s.dim;
    a.vdim = s.vdim;
    a.taps = s.taps;
    a.a_rank = s.a1.rows;
    a.g_rank = s.g1.rows;
    a.ld = pad_to(w.in.rows, 4);
    if (s.a2.rows != hd || s.a2.cols != s.a1.rows || s.g2.rows != vd || s.g2.cols != s.g1.rows || !s.a2.data || !s.g2.data)
        return ZQ_ERR_BAD_ARG;
    RUN(L.put(&a.low, hd + vd, rank));
    RUN(L.rows_cut(a.low, s.a2, 0));
    RUN(L.rows_cut(a.low, s.g2, hd));
    RUN(L.send(&a.low));
    float *conv, *A_log, *dt_bias, *norm;
    RUN(L.vec(&conv, s.conv, (size_t)ch * s.taps));
    RUN(L.vec(&A_log, s.A_log, H));
    RUN(L.vec(&dt_bias, s.dt_bias, hd));
    RUN(L.vec(&norm, s.mix_norm, s.vdim));
    a.conv = conv;
    a.A_log = A_log;
    a.dt_bias = dt_bias;
    a.norm = norm;
    a.eps = m->c.norm_eps;
    a.out_pitch = w.o.kp;
    RUN(slot_state(m, &a.S, (size_t)hd * s.vdim, L.st));
    return zeroed(m, reinterpret_cast<void**>(&a.ring), (size_t)m->c.n_seq * s.taps * ch * sizeof(float), L.st);
}

int load_latent(zq_decoder* m, Loader& L, Layer& d, const zq_decoder_layer& s, uint32_t index) {
    if (!s.heads || !s.dim || !s.vdim || !s.kv_rank || s.rot_dim % 2 || !(s.rot_base > 0.0f)) return ZQ_ERR_BAD_ARG;
    LatentLayer& w = d.lat;
    const uint32_t H = s.heads, kd = H * s.dim, vd = H * s.vdim, qd = H * (s.dim + s.rot_dim);
    w.s = LatentShape{H, s.dim, s.rot_dim, s.vdim, s.kv_rank, pad_to(s.kv_rank + s.rot_dim, 16), m->c.ctx, m->c.n_seq};
    w.scale = s.scale;
    w.own = s.kv_from < 0;
    RUN(stack(L, d, s, &w.in, {{&s.q, qd}, {&s.dkv, w.own ? s.kv_rank + s.rot_dim : 0}}));
    RUN(L.matrix(&w.o, s.o, m->c.width, vd));
    RUN(L.put(&w.up, kd + vd, s.kv_rank));
    RUN(L.rows_from(w.up, s.uk, kd, 0));
    RUN(L.rows_from(w.up, s.uv, vd, kd));
    RUN(L.send(&w.up));
    std::vector<float> freq(s.rot_dim / 2 + 1, 0.0f);
    for (uint32_t i = 0; i < s.rot_dim / 2; ++i) freq[i] = (float)pow((double)s.rot_base, -2.0 * i / s.rot_dim);
    RUN(L.vec(&w.freq, freq.data(), freq.size()));
    ZQ_CUDA(cudaStreamSynchronize(L.st));  // `freq` goes
    if (w.own) {
        RUN(L.vec(&w.norm, s.dkv_norm, s.kv_rank));
        return zeroed(m, &w.cache, (size_t)m->c.n_seq * m->c.ctx * w.s.keyp * act_bytes(m->f32), L.st);
    }
    if ((uint32_t)s.kv_from >= index) return ZQ_ERR_BAD_ARG;
    const Layer& from = m->layers[s.kv_from];
    if (from.mixer != ZQ_MIXER_LATENT || !from.lat.own || from.lat.s.rank != s.kv_rank || from.lat.s.rot != s.rot_dim)
        return ZQ_ERR_BAD_ARG;
    w.cache = from.lat.cache;
    return ZQ_OK;
}

int load_attention(zq_decoder* m, Loader& L, Layer& d, const zq_decoder_layer& s, GqaShape* first) {
    const uint32_t E = m->c.width;
    if (!s.heads || !s.kv_heads || s.heads % s.kv_heads || !s.dim || !s.vdim) return ZQ_ERR_BAD_ARG;
    AttentionLayer& a = d.att;
    a.s = GqaShape{s.heads, s.kv_heads, s.dim, s.vdim, pad_to(s.dim, 16), pad_to(s.vdim, 16), m->c.ctx, m->c.n_seq};
    a.scale = s.scale;
    a.temp_coef = s.q_temp_coef;
    a.temp_every = s.q_temp_every;
    const uint32_t qd = s.heads * s.dim, kd = s.kv_heads * s.dim, vd = s.kv_heads * s.vdim;
    RUN(L.put(&a.qkv, qd + kd + vd, E));
    RUN(L.rows_from(a.qkv, s.q, qd, 0));
    RUN(L.rows_from(a.qkv, s.k, kd, qd));
    RUN(L.rows_from(a.qkv, s.v, vd, qd + kd));
    RUN(L.send(&a.qkv));
    RUN(L.matrix(&a.o, s.o, E, s.heads * s.vdim));
    RUN(L.vec(&a.q_norm, s.q_norm, s.dim));
    RUN(L.vec(&a.k_norm, s.k_norm, s.dim));
    if (s.v_mix) {
        a.v_mix = true;
        a.v_first = first->kv_heads == 0;
        if (a.v_first) {
            *first = a.s;
        } else {
            if (s.kv_heads != first->kv_heads || s.vdim != first->vdim) return ZQ_ERR_UNSUPPORTED;  // nothing to mix with
            RUN(L.vec(&a.vmix, &s.vmix, 1));
        }
    }
    const size_t rows = (size_t)m->c.n_seq * m->c.ctx * s.kv_heads;
    RUN(zeroed(m, &a.kc, rows * a.s.dimp * act_bytes(m->f32), L.st));
    return zeroed(m, &a.vc, rows * a.s.vdimp * act_bytes(m->f32), L.st);
}

int load_wkv(zq_decoder* m, Loader& L, Layer& d, const zq_decoder_layer& s) {
    const uint32_t E = m->c.width, hd = s.heads * s.dim;
    if (!s.heads || !s.dim || !s.decay_rank) return ZQ_ERR_BAD_ARG;
    if (s.dim > 256) return ZQ_ERR_LIMIT;
    WkvLayer& w = d.wkv;
    w.heads = s.heads;
    w.dim = s.dim;
    w.rank = s.decay_rank;
    RUN(L.put(&w.in, 4 * hd + s.decay_rank, E));
    RUN(L.rows_from(w.in, s.r, hd, 0));
    RUN(L.rows_from(w.in, s.k, hd, hd));
    RUN(L.rows_from(w.in, s.v, hd, 2 * hd));
    RUN(L.rows_from(w.in, s.g, hd, 3 * hd));
    RUN(L.rows_from(w.in, s.w1, s.decay_rank, 4 * hd));
    RUN(L.send(&w.in));
    RUN(L.matrix(&w.w2, s.w2, hd, s.decay_rank));
    RUN(L.matrix(&w.o, s.o, E, hd));
    RUN(L.vec(&w.mu, s.mu, (size_t)5 * E));
    RUN(L.vec(&w.w0, s.w0, hd));
    RUN(L.vec(&w.u, s.u, hd));
    RUN(L.vec(&w.norm, s.mix_norm, hd));
    RUN(slot_state(m, &w.state, (size_t)hd * s.dim, L.st));
    return slot_state(m, &w.prev, E, L.st);
}

GluSpec glu_spec(uint32_t kind, float limit) {
    GluSpec g;
    g.kind = kind == ZQ_GLU_CLAMPED ? GLU_CLAMPED : GLU_SILU;
    g.limit = limit;
    return g;
}

int load_moe(zq_decoder* m, Loader& L, Layer& d, const zq_decoder_layer& s) {
    const uint32_t E = m->c.width;
    if (!s.experts || !s.top || s.top > s.experts || !s.expert_ff || !s.expert_gate || !s.expert_up || !s.expert_down)
        return ZQ_ERR_BAD_ARG;
    if (s.experts > 1024) return ZQ_ERR_LIMIT;
    MoeWeights& w = d.moe;
    w.experts = s.experts;
    w.top = s.top;
    w.width = E;
    w.ffp = pad64(s.expert_ff);
    RUN(L.put(&w.gate_up, s.experts * 2 * w.ffp, E));
    for (uint32_t e = 0; e < s.experts; ++e) {
        RUN(L.glu_from(w.gate_up, s.expert_gate[e], s.expert_ff, e * 2 * w.ffp, false));
        RUN(L.glu_from(w.gate_up, s.expert_up[e], s.expert_ff, e * 2 * w.ffp, true));
    }
    RUN(L.send(&w.gate_up));
    RUN(L.put(&w.down, s.experts * E, s.expert_ff));
    for (uint32_t e = 0; e < s.experts; ++e) RUN(L.rows_from(w.down, s.expert_down[e], E, e * E));
    RUN(L.send(&w.down));
    if (s.route > ZQ_ROUTE_SOFTMAX || s.expert_glu > ZQ_GLU_CLAMPED || s.shared_glu > ZQ_GLU_CLAMPED) return ZQ_ERR_UNSUPPORTED;
    d.shared_gated = s.shared_sg.data != nullptr;
    if (d.shared_gated && !s.shared_ff) return ZQ_ERR_BAD_ARG;
    d.route_kind = s.route == ZQ_ROUTE_SOFTMAX ? ROUTE_SOFTMAX : ROUTE_SIGMOID;
    w.scale_input = d.route_kind == ROUTE_SIGMOID;
    w.glu = glu_spec(s.expert_glu, s.expert_limit);
    w.shared_glu = glu_spec(s.shared_glu, s.shared_limit);
    if (s.router_bias) RUN(L.vec(&d.router_bias, s.router_bias, s.experts));
    if (d.router_col < 0) {
        RUN(L.put(&d.router, s.experts + (d.shared_gated ? 1 : 0), E));
        RUN(put_router(L, d.router, s, 0));
        RUN(L.send(&d.router));
    }
    if (s.shared_ff) {
        w.shared_ffp = pad64(s.shared_ff);
        RUN(L.glu(&w.shared_gate_up, s.shared_gate, s.shared_up, s.shared_ff, E));
        RUN(L.matrix(&w.shared_down, s.shared_down, E, s.shared_ff));
    }
    return ZQ_OK;
}

int load(zq_decoder* m, const zq_decoder_weights* w, cudaStream_t st) {
    const zq_decoder_config& C = m->c;
    const uint32_t E = C.width;
    Loader L{m, st, {}};
    RUN(L.matrix(&m->embed, w->embed, C.vocab, E));
    if (w->head.data)
        RUN(L.matrix(&m->head, w->head, C.vocab, E));
    else
        m->head = m->embed;
    if (w->embed_norm) RUN(L.vec(&m->embed_norm, w->embed_norm, E));
    RUN(L.vec(&m->final_norm, w->final_norm, E));
    m->layers.resize(C.layers);
    GqaShape first{};  // of the first layer whose values later ones mix in
    for (uint32_t l = 0; l < C.layers; ++l) {
        const zq_decoder_layer& s = w->layers[l];
        Layer& d = m->layers[l];
        d.mixer = s.mixer;
        d.mlp = s.mlp;
        d.parallel = s.parallel != 0;
        if (s.mlp > ZQ_MLP_MOE) return ZQ_ERR_UNSUPPORTED;
        RUN(L.vec(&d.norm1, s.norm1, E));
        if (!d.parallel) RUN(L.vec(&d.norm1b, s.norm1b, E));
        switch (s.mixer) {
            case ZQ_MIXER_ATTENTION: RUN(load_attention(m, L, d, s, &first)); break;
            case ZQ_MIXER_WKV: RUN(load_wkv(m, L, d, s)); break;
            case ZQ_MIXER_MEMORY: RUN(load_memory(m, L, d, s)); break;
            case ZQ_MIXER_DELTA: RUN(load_delta(m, L, d, s)); break;
            case ZQ_MIXER_LATENT: RUN(load_latent(m, L, d, s, l)); break;
            default: return ZQ_ERR_UNSUPPORTED;
        }
        if (s.mlp != ZQ_MLP_NONE && !d.parallel) {
            RUN(L.vec(&d.norm2, s.norm2, E));
            RUN(L.vec(&d.norm2b, s.norm2b, E));
        }
        if (s.mlp == ZQ_MLP_DENSE) {
            if (!s.ff) return ZQ_ERR_BAD_ARG;
            if (s.mlp_glu > ZQ_GLU_CLAMPED) return ZQ_ERR_UNSUPPORTED;
            d.glu = glu_spec(s.mlp_glu, s.limit);
            RUN(L.glu(&d.gate_up, s.gate, s.up, s.ff, E));
            RUN(L.matrix(&d.down, s.down, E, s.ff));
        } else if (s.mlp == ZQ_MLP_MOE) {
            RUN(load_moe(m, L, d, s));
        }
    }

    // scratch: a prefill piece of up to max_rows tokens, or one row per sequence
    m->hp = pad64(E);
    m->max_rows = std::max(std::min(C.ctx, 2048u), C.n_seq);
    const size_t R = m->max_rows, ab = act_bytes(m->f32);
    size_t proj = 0, q = 0, att = 0, hid = 0, parts = 0, pairs = 0, z = 0, experts = 0, decay = 0, chunk = 0, work = 0;
    bool wkv = false, y2 = false;
    auto mixer_room = [&](const DenseWeight& in, const DenseWeight& o, size_t bytes) {
        proj = std::max(proj, (size_t)pad_to(in.rows, 4));
        att = std::max(att, (size_t)o.kp);
        work = std::max(work, bytes);
    };
    for (const Layer& d : m->layers) {
        y2 = y2 || (d.parallel && d.mlp == ZQ_MLP_DENSE);
        if (d.mixer == ZQ_MIXER_ATTENTION) {
            const GqaShape& s = d.att.s;
            mixer_room(d.att.qkv, d.att.o, gqa_work_bytes(s, C.n_seq));
            q = std::max(q, (size_t)s.heads * s.dimp);
        } else if (d.mixer == ZQ_MIXER_MEMORY) {
            mixer_room(d.mem.in, d.mem.o, memory_work_floats(d.mem.heads, d.mem.dim, d.mem.vdim, m->max_rows) * sizeof(float));
        } else if (d.mixer == ZQ_MIXER_DELTA) {
            mixer_room(d.delta.in, d.delta.o, delta_work_floats(d.delta.args, m->max_rows) * sizeof(float));
        } else if (d.mixer == ZQ_MIXER_LATENT) {
            mixer_room(d.lat.in, d.lat.o, latent_work_bytes(d.lat.s, m->max_rows, m->f32));
        } else {
            wkv = true;
            mixer_room(d.wkv.in, d.wkv.o, 0);
            decay = std::max(decay, (size_t)d.wkv.heads * d.wkv.dim);
            chunk = std::max(chunk, wkv_chunk_floats(d.wkv.heads, d.wkv.dim, m->max_rows));
        }
        if (d.mlp == ZQ_MLP_DENSE) hid = std::max(hid, R * d.down.kp);
        if (d.mlp == ZQ_MLP_MOE) {
            const MoeWeights& w2 = d.moe;
            const size_t np = R * w2.top;
            if (np / 32 + w2.experts > kMoeMaxTiles) return ZQ_ERR_LIMIT;
            pairs = std::max(pairs, np);
            hid = std::max(hid, np * w2.ffp + R * w2.shared_ffp);
            parts = std::max(parts, (np + R) * E);
            if (d.router_col < 0) z = std::max(z, R * d.router.rows);
            experts = std::max(experts, (size_t)w2.experts);
        }
    }
    DeviceArena& A = m->arena;
    RUN(A.alloc_n(&m->x, R * E));
    // y: room for the addends of a product whose K is cut, up to 64 MB of them
    m->y_floats = std::max(R * E, std::min(8 * R * E, (size_t)16 << 20));
    RUN(A.alloc_n(&m->y, m->y_floats));
    if (y2) RUN(A.alloc_n(&m->y2, m->y_floats));
    RUN(A.alloc(&m->h, R * m->hp * ab));
    RUN(A.alloc_n(&m->proj, R * proj));
    RUN(A.alloc(&m->q, R * q * ab));
    RUN(A.alloc(&m->att, R * att * ab));
    RUN(A.alloc(&m->hid, hid * ab));
    RUN(zeroed(m, &m->work, work, st));
    if (first.kv_heads) RUN(A.alloc_n(&m->v_first, R * first.kv_heads * first.vdim));
    if (wkv) {
        RUN(A.alloc_n(&m->h32, R * E));
        RUN(A.alloc(&m->mix, 5 * R * m->hp * ab));
        RUN(A.alloc_n(&m->decay, R * decay));
        RUN(A.alloc_n(&m->chunk, chunk));
    }
    if (pairs) {
        RUN(A.alloc_n(&m->parts, parts));
        RUN(A.alloc_n(&m->z, z));
        RUN(A.alloc_n(&m->xs, m->f32 ? 4 : pairs * m->hp));
        RUN(A.alloc_n(&m->route.ids, pairs));
        RUN(A.alloc_n(&m->route.weights, pairs));
        RUN(A.alloc_n(&m->route.place, pairs));
        RUN(A.alloc_n(&m->route.source, pairs));
        RUN(A.alloc_n(&m->route.offsets, experts + 1));
        RUN(A.alloc_n(&m->route.tiles, (size_t)2 * kMoeMaxTiles + 1));
    }
    RUN(A.alloc_n(&m->logits, (size_t)C.n_seq * C.vocab));
    RUN(A.alloc_n(&m->d_tokens, R));
    RUN(A.alloc_n(&m->d_pos, R));
    RUN(A.alloc_n(&m->d_slots, R));
    RUN(A.alloc_n(&m->d_want, R));
    RUN(A.alloc_n(&m->d_arg, 1));
    RUN(A.alloc_n(&m->d_rec, 1));
    RUN(A.alloc_n(&m->d_record, C.ctx));
    m->seq_lens.assign(C.n_seq, 0);
    for (const Layer& d : m->layers) {
        if (m->side || !d.parallel || d.mlp == ZQ_MLP_NONE) continue;
        ZQ_CUDA(cudaStreamCreateWithFlags(&m->side, cudaStreamNonBlocking));
        ZQ_CUDA(cudaEventCreateWithFlags(&m->forked, cudaEventDisableTiming));
        ZQ_CUDA(cudaEventCreateWithFlags(&m->joined, cudaEventDisableTiming));
    }
    ZQ_CUDA(cudaStreamSynchronize(st));  // host tensors may be released
    return ZQ_OK;
}

// ------------------------------------------------------------------------------------------------ forward pass
struct Pass {
    uint32_t rows;
    bool one_sequence;     // consecutive tokens of slot d_slots[0]; otherwise row r is a token of slot d_slots[r]
    uint32_t pos0;         // one_sequence with several rows: position of row 0
    bool all_logits;       // decode: logits of every row to m->logits
    uint32_t n_want;       // otherwise: of the rows d_want[0 .. n_want) to want_out
    float* want_out;
    bool greedy;
    uint32_t trail_at;     // first row of the trail that this pass writes
    uint32_t slot;         // one_sequence with several rows: its slot
};

// What follows the residual sum of a layer: the norm ahead of the next mixer (with its token shift), or the last norm.
void set_next(zq_decoder* m, const Pass& P, uint32_t next, AddNormArgs& a) {
    if (next < m->layers.size()) {
        const Layer& d = m->layers[next];
        a.pre_w = d.norm1;
        if (d.mixer != ZQ_MIXER_WKV || d.parallel) a.h = m->h;
        if (d.mixer != ZQ_MIXER_WKV) return;
        if (P.one_sequence && P.rows > 1) {
            a.h32 = m->h32;
        } else {
            a.mu = d.wkv.mu;
            a.prev = d.wkv.prev;
            a.slots = m->d_slots;
            a.mix = m->mix;
            a.n_mix = 5;
            a.mix_rows = m->max_rows;
        }
    } else if (P.all_logits) {
        a.pre_w = m->final_norm;
        a.h = m->h;
    }
}

AddNormArgs norm_args(const zq_decoder* m) {
    AddNormArgs a{};
    a.x = m->x;
    a.width = m->c.width;
    a.hp = m->hp;
    a.eps = m->c.norm_eps;
    return a;
}

int attention(zq_decoder* m, const AttentionLayer& a, const Pass& P, cudaStream_t st) {
    RUN(launch_dense_linear(a.qkv, one_group(a.qkv.rows), m->h, m->max_rows, P.rows, m->proj, a.qkv.rows, m->f32, st));
    QkvPostArgs q{};
    q.s = a.s;
    q.qkv = m->proj;
    q.q_norm = a.q_norm;
    q.k_norm = a.k_norm;
    q.eps = m->c.norm_eps;
    q.temp_coef = a.temp_coef;
    q.temp_every = a.temp_every;
    q.vmix = a.vmix;
    q.v_first = a.v_mix ? m->v_first : nullptr;
    q.q = m->q;
    q.kc = a.kc;
    q.vc = a.vc;
    q.pos = m->d_pos;
    q.slots = m->d_slots;
    RUN(launch_gqa_layer(q, m->att, a.o.kp, a.scale, P.rows, P.one_sequence, P.pos0, m->work, m->f32, st));
    return launch_dense_linear(a.o, one_group(a.o.rows), m->att, m->max_rows, P.rows, m->y, m->c.width, m->f32, st, &m->y_add,
                               m->y_floats);
}

int wkv(zq_decoder* m, const WkvLayer& w, const Pass& P, cudaStream_t st) {
    const bool piece = P.one_sequence && P.rows > 1;
    const uint32_t hd = w.heads * w.dim;
    if (piece)
        RUN(launch_token_shift(m->h32, w.mu, w.prev, m->d_slots, 5, P.rows, m->max_rows, m->c.width, m->mix, m->f32, st));
    LinGroups G{};
    G.n = 5;
    for (uint32_t i = 0; i < 5; ++i) G.g[i] = LinGroup{i * hd, i < 4 ? hd : w.rank, i * m->max_rows, i * hd};
    const uint32_t ld = pad_to(w.in.rows, 4);  // 16-byte rows for the recurrence's copies
    RUN(launch_dense_linear(w.in, G, m->mix, 5 * m->max_rows, P.rows, m->proj, ld, m->f32, st));
    WkvArgs a{};
    a.heads = w.heads;
    a.dim = w.dim;
    a.rank = w.rank;
    a.rank_p = w.w2.kp;
    a.ld = ld;
    a.rkvg = m->proj;
    a.w2 = w.w2.w;
    a.w0 = w.w0;
    a.u = w.u;
    a.norm = w.norm;
    a.eps = m->c.norm_eps;
    a.state = w.state;
    a.slots = m->d_slots;
    a.out = m->att;
    a.out_pitch = w.o.kp;
    a.h32 = piece ? m->h32 : nullptr;
    a.prev = w.prev;
    a.width = m->c.width;
    a.decay = m->decay;
    a.chunk = m->chunk;
    RUN(launch_wkv(a, P.rows, P.one_sequence, m->f32, st));
    return launch_dense_linear(w.o, one_group(w.o.rows), m->att, m->max_rows, P.rows, m->y, m->c.width, m->f32, st, &m->y_add,
                               m->y_floats);
}

// The products around a mixer of the kinds below: its first one (with the router's logits; the other kinds have theirs
// inside) and its last one.
int mixer_in(zq_decoder* m, const Layer& d, const Pass& P, cudaStream_t st) {
    const DenseWeight* in = nullptr;
    if (d.mixer == ZQ_MIXER_MEMORY) in = &d.mem.in;
    if (d.mixer == ZQ_MIXER_DELTA) in = &d.delta.in;
    if (d.mixer == ZQ_MIXER_LATENT) in = &d.lat.in;
    if (!in) return ZQ_OK;
    return launch_dense_linear(*in, one_group(in->rows), m->h, m->max_rows, P.rows, m->proj, pad_to(in->rows, 4), m->f32, st);
}
int mixer_out(zq_decoder* m, const DenseWeight& o, const Pass& P, cudaStream_t st) {
    return launch_dense_linear(o, one_group(o.rows), m->att, m->max_rows, P.rows, m->y, m->c.width, m->f32, st, &m->y_add,
                               m->y_floats);
}

int memory(zq_decoder* m, const MemoryLayer& w, const Pass& P, cudaStream_t st) {
    MemoryArgs a{};
    a.heads = w.heads;
    a.dim = w.dim;
    a.vdim = w.vdim;
    a.ld = pad_to(w.in.rows, 4);
    a.in = m->proj;
    a.i_bias = w.i_bias;
    a.f_bias = w.f_bias;
    a.gate_cap = w.gate_cap;
    a.norm = w.norm;
    a.eps = m->c.norm_eps;
    a.S = w.S;
    a.n = w.n;
    a.m = w.m;
    a.slots = m->d_slots;
    a.out = m->att;
    a.out_pitch = w.o.kp;
    a.work = static_cast<float*>(m->work);
    RUN(launch_memory(a, P.rows, P.one_sequence, m->f32, st));
    return mixer_out(m, w.o, P, st);
}

int delta(zq_decoder* m, const DeltaLayer& w, const Pass& P, cudaStream_t st) {
    DeltaArgs a = w.args;
    a.in = m->proj;
    a.pos = m->d_pos;
    a.slots = m->d_slots;
    a.out = m->att;
    a.work = static_cast<float*>(m->work);
    a.max_rows = m->max_rows;
    RUN(launch_delta(a, P.rows, P.one_sequence, m->f32, st));
    return mixer_out(m, w.o, P, st);
}

int latent(zq_decoder* m, const LatentLayer& w, const Pass& P, cudaStream_t st) {
    LatentArgs a{};
    a.s = w.s;
    a.in = m->proj;
    a.ld = pad_to(w.in.rows, 4);
    a.own = w.own;
    a.norm = w.norm;
    a.eps = m->c.norm_eps;
    a.scale = w.scale;
    a.freq = w.freq;
    a.up = w.up;
    a.cache = w.cache;
    a.pos = m->d_pos;
    a.slots = m->d_slots;
    a.slot0 = P.slot;
    a.out = m->att;
    a.out_pitch = w.o.kp;
    a.work = m->work;
    a.max_rows = m->max_rows;
    RUN(launch_latent(a, P.rows, P.one_sequence, P.pos0, m->f32, st));
    return mixer_out(m, w.o, P, st);
}

int mixer(zq_decoder* m, const Layer& d, const Pass& P, cudaStream_t st) {
    switch (d.mixer) {
        case ZQ_MIXER_ATTENTION: return attention(m, d.att, P, st);
        case ZQ_MIXER_WKV: return wkv(m, d.wkv, P, st);
        case ZQ_MIXER_MEMORY: return memory(m, d.mem, P, st);
        case ZQ_MIXER_DELTA: return delta(m, d.delta, P, st);
        default: return latent(m, d.lat, P, st);
    }
}

int experts(zq_decoder* m, const Layer& d, const Pass& P, AddNormArgs& next, cudaStream_t st) {
    const MoeWeights& w = d.moe;
    const uint32_t T = P.rows, pairs = T * w.top;
    const float* z = m->z;
    uint32_t ld = d.router.rows;
    if (d.router_col >= 0) {
        z = m->proj + d.router_col;
        ld = pad_to((uint32_t)d.router_col + w.experts + (d.shared_gated ? 1 : 0), 4);
    } else {
        RUN(launch_dense_linear(d.router, one_group(d.router.rows), m->h, m->max_rows, T, m->z, ld, m->f32, st));
    }
    RUN(launch_route(z, ld, w.experts, w.top, d.router_bias, d.route_kind, m->route, T, st));
    next.parts = m->parts;
    next.top = w.top;
    if (!w.scale_input) next.part_w = m->route.weights;
    float* shared = m->parts + (size_t)pairs * w.width;
    if (w.shared_ffp) {
        next.shared = shared;
        if (d.shared_gated) {
            next.shared_gate = z + w.experts;
            next.gate_stride = ld;
        }
    }
    if (m->f32 || T < kDenseGemmMinRows) return launch_moe_pairs(w, m->route, m->h, T, m->hid, m->parts, m->f32, st);
    uint32_t bn = 32;
    while (bn < 256 && bn * w.experts < pairs) bn <<= 1;
    RUN(launch_moe_plan(m->route, w.experts, w.top, T, bn, static_cast<const bf16*>(m->h), m->hp, w.scale_input, m->xs, st));
    bf16* hid = static_cast<bf16*>(m->hid);
    RUN(launch_moe_grouped(w, m->route, m->xs, T, bn, hid, m->parts, st));
    next.place = m->route.place;
    if (w.shared_ffp) {
        bf16* hs = hid + (size_t)pairs * w.ffp;
        RUN(launch_dense_glu(w.shared_gate_up, m->h, T, hs, w.shared_glu, false, st));
        RUN(launch_dense_linear(w.shared_down, one_group(w.width), hs, T, T, shared, w.width, false, st));
    }
    return ZQ_OK;
}

// What a layer's feed-forward part makes of m->h; `next` learns where its output lies.
int feed_forward(zq_decoder* m, const Layer& d, const Pass& P, AddNormArgs& next, cudaStream_t st) {
    if (d.mlp == ZQ_MLP_MOE) return experts(m, d, P, next, st);
    float* y = d.parallel ? m->y2 : m->y;
    Addends add;
    RUN(launch_dense_glu(d.gate_up, m->h, P.rows, m->hid, d.glu, m->f32, st));
    RUN(launch_dense_linear(d.down, one_group(d.down.rows), m->hid, P.rows, P.rows, y, m->c.width, m->f32, st, &add, m->y_floats));
    (d.parallel ? next.y2 : next.y) = y;
    (d.parallel ? next.y2_add : next.y_add) = add;
    return ZQ_OK;
}

// The feed-forward part on the side stream, from what st has reached.
int feed_forward_beside(zq_decoder* m, const Layer& d, const Pass& P, AddNormArgs& next, cudaStream_t st) {
    ZQ_CUDA(cudaEventRecord(m->forked, st));
    ZQ_CUDA(cudaStreamWaitEvent(m->side, m->forked, 0));
    whole_dependency = true;
    const int rc = feed_forward(m, d, P, next, m->side);
    whole_dependency = false;
    RUN(rc);
    ZQ_CUDA(cudaEventRecord(m->joined, m->side));
    return ZQ_OK;
}

int forward(zq_decoder* m, const Pass& P, cudaStream_t st) {
    if (P.rows == 0 || P.rows > m->max_rows) return ZQ_ERR_BAD_ARG;
    AddNormArgs a = norm_args(m);
    a.embed = m->embed.w;
    a.embed_kp = m->embed.kp;
    a.embed_scale = m->c.embed_scale;
    a.embed_w = m->embed_norm;
    a.tokens = m->d_tokens;
    set_next(m, P, 0, a);
    RUN(launch_add_norm(a, P.rows, m->f32, st));
    for (uint32_t l = 0; l < m->layers.size(); ++l) {
        const Layer& d = m->layers[l];
        a = norm_args(m);
        a.post_w = d.norm1b;
        const bool ff = d.mlp != ZQ_MLP_NONE, beside = ff && d.parallel && P.rows < kDenseGemmMinRows;
        if (beside && d.router_col < 0) RUN(feed_forward_beside(m, d, P, a, st));  // otherwise the first product has the router's logits
        RUN(mixer_in(m, d, P, st));
        if (beside && d.router_col >= 0) RUN(feed_forward_beside(m, d, P, a, st));
        RUN(mixer(m, d, P, st));
        a.y = m->y;
        a.y_add = m->y_add;
        if (beside) {
            ZQ_CUDA(cudaStreamWaitEvent(st, m->joined, 0));
            whole_dependency = true;
        } else if (ff) {
            if (!d.parallel) {
                a.pre_w = d.norm2;
                a.h = m->h;
                RUN(launch_add_norm(a, P.rows, m->f32, st));
                a = norm_args(m);
                a.post_w = d.norm2b;
            }
            RUN(feed_forward(m, d, P, a, st));
        }
        set_next(m, P, l + 1, a);
        RUN(launch_add_norm(a, P.rows, m->f32, st));
        if (m->trail && P.trail_at < m->trail_rows) {
            const uint32_t n = std::min(P.rows, m->trail_rows - P.trail_at);
            ZQ_CUDA(cudaMemcpyAsync(m->trail + ((size_t)l * m->trail_rows + P.trail_at) * m->c.width, m->x,
                                    (size_t)n * m->c.width * sizeof(float), cudaMemcpyDeviceToDevice, st));
        }
    }
    if (P.all_logits) {
        RUN(launch_dense_linear(m->head, one_group(m->head.rows), m->h, m->max_rows, P.rows, m->logits, m->c.vocab, m->f32, st));
    } else if (P.n_want) {
        a = norm_args(m);
        a.pre_w = m->final_norm;
        a.h = m->h;
        a.rows_from = m->d_want;
        RUN(launch_add_norm(a, P.n_want, m->f32, st));
        RUN(launch_dense_linear(m->head, one_group(m->head.rows), m->h, m->max_rows, P.n_want, P.want_out, m->c.vocab, m->f32, st));
    }
    if (P.greedy) {
        RUN(zq_argmax(m->logits, m->c.vocab, m->d_arg, st));
        feed_row_kernel<<<1, 1, 0, st>>>(m->d_tokens, m->d_pos, m->d_rec, m->d_arg, m->d_record);
        ZQ_LAUNCH_CHECK();
    }
    return ZQ_OK;
}

// One token of the sequence whose slot, token and position are set in row 0: recorded on first use, then replayed.
int step(zq_decoder* m, int variant, uint32_t trail_at, cudaStream_t st) {
    Pass P{1, true, 0, variant != STEP_CACHE_ONLY, 0, nullptr, variant == STEP_GREEDY, trail_at, 0};
    if (m->trail) return forward(m, P, st);
    return m->graphs.run(variant, st, [&](cudaStream_t s) { return forward(m, P, s); });
}

int set_row(zq_decoder* m, uint32_t seq, uint32_t token, cudaStream_t st) {
    set_row_kernel<<<1, 1, 0, st>>>(m->d_tokens, m->d_pos, m->d_slots, m->d_rec, token, m->seq_lens[seq], seq);
    ZQ_LAUNCH_CHECK();
    return ZQ_OK;
}

}  // namespace

extern "C" {

int zq_decoder_create(const zq_decoder_config* cfg, const zq_decoder_weights* w, zq_stream stream, zq_decoder** out) {
    if (!cfg || !w || !out || !w->layers) return ZQ_ERR_BAD_ARG;
    *out = nullptr;
    if (!cfg->vocab || !cfg->width || !cfg->layers || !cfg->ctx || !cfg->n_seq || cfg->n_seq > 1024 ||
        (cfg->precision != ZQ_PRECISION_BF16 && cfg->precision != ZQ_PRECISION_F32))
        return ZQ_ERR_BAD_ARG;
    if (cfg->width > 12288) return ZQ_ERR_LIMIT;
    zq_decoder* m = new (std::nothrow) zq_decoder;
    if (!m) return ZQ_ERR_NO_MEM;
    m->c = *cfg;
    m->f32 = cfg->precision == ZQ_PRECISION_F32;
    int rc;
    try {
        rc = load(m, w, as_stream(stream));
    } catch (const std::bad_alloc&) {
        rc = ZQ_ERR_NO_MEM;
    }
    if (rc != ZQ_OK) {
        delete m;
        return rc;
    }
    *out = m;
    return ZQ_OK;
}

int zq_decoder_free(zq_decoder* m) {
    delete m;
    return ZQ_OK;
}

int zq_decoder_reset_seq(zq_decoder* m, uint32_t seq, zq_stream stream) {
    if (!m || seq >= m->c.n_seq) return ZQ_ERR_BAD_ARG;
    cudaStream_t st = as_stream(stream);
    for (const SlotState& x : m->states) ZQ_CUDA(cudaMemsetAsync(x.base + seq * x.bytes, 0, x.bytes, st));
    m->seq_lens[seq] = 0;
    return ZQ_OK;
}

int zq_decoder_reset_cache(zq_decoder* m, zq_stream stream) {
    if (!m) return ZQ_ERR_BAD_ARG;
    for (uint32_t s = 0; s < m->c.n_seq; ++s) {
        if (m->seq_lens[s] == 0) continue;
        const int rc = zq_decoder_reset_seq(m, s, stream);
        if (rc != ZQ_OK) return rc;
    }
    return ZQ_OK;
}

int zq_decoder_seq_len_of(const zq_decoder* m, uint32_t seq, uint32_t* seq_len) {
    if (!m || !seq_len || seq >= m->c.n_seq) return ZQ_ERR_BAD_ARG;
    *seq_len = m->seq_lens[seq];
    return ZQ_OK;
}

int zq_decoder_extend(zq_decoder* m, uint32_t seq, const uint32_t* h_tokens, uint32_t n, const uint32_t* h_want,
                      uint32_t n_want, float* d_out, zq_stream stream) {
    if (!m || !h_tokens || seq >= m->c.n_seq || (n_want && (!h_want || !d_out))) return ZQ_ERR_BAD_ARG;
    if (n == 0 || n > m->c.ctx - m->seq_lens[seq]) return ZQ_ERR_SEQUENCE;
    for (uint32_t t = 0; t < n; ++t)
        if (h_tokens[t] >= m->c.vocab) return ZQ_ERR_BAD_ARG;
    for (uint32_t i = 0; i < n_want; ++i)
        if (h_want[i] >= n || (i && h_want[i] <= h_want[i - 1])) return ZQ_ERR_BAD_ARG;
    cudaStream_t st = as_stream(stream);
    const size_t V = m->c.vocab;
    std::vector<int32_t> want;
    uint32_t w = 0;
    for (uint32_t t0 = 0; t0 < n; t0 += m->max_rows) {
        const uint32_t T = std::min(n - t0, m->max_rows), w0 = w;
        want.clear();
        for (; w < n_want && h_want[w] < t0 + T; ++w) want.push_back((int32_t)(h_want[w] - t0));
        int rc;
        if (T == 1) {
            if ((rc = set_row(m, seq, h_tokens[t0], st)) != ZQ_OK) return rc;
            if ((rc = step(m, want.empty() ? STEP_CACHE_ONLY : STEP_LOGITS, t0, st)) != ZQ_OK) return rc;
            if (!want.empty())
                ZQ_CUDA(cudaMemcpyAsync(d_out + w0 * V, m->logits, V * sizeof(float), cudaMemcpyDeviceToDevice, st));
        } else {
            set_rows_kernel<<<(T + 255) / 256, 256, 0, st>>>(m->d_pos, m->d_slots, m->seq_lens[seq], seq, T);
            ZQ_LAUNCH_CHECK();
            ZQ_CUDA(cudaMemcpyAsync(m->d_tokens, h_tokens + t0, T * sizeof(uint32_t), cudaMemcpyHostToDevice, st));
            if (!want.empty())
                ZQ_CUDA(cudaMemcpyAsync(m->d_want, want.data(), want.size() * sizeof(int32_t), cudaMemcpyHostToDevice, st));
            Pass P{T, true, m->seq_lens[seq], false, (uint32_t)want.size(), d_out + w0 * V, false, t0, seq};
            if ((rc = forward(m, P, st)) != ZQ_OK) return rc;
            ZQ_CUDA(cudaStreamSynchronize(st));  // the host arrays are the caller's, or change with the next piece
        }
        m->seq_lens[seq] += T;
    }
    return ZQ_OK;
}

int zq_decoder_prefill_seq(zq_decoder* m, uint32_t seq, const uint32_t* h_tokens, uint32_t n, zq_stream stream,
                           const float** d_logits) {
    if (!m || !h_tokens || !d_logits || seq >= m->c.n_seq) return ZQ_ERR_BAD_ARG;
    if (n == 0 || n > m->c.ctx) return ZQ_ERR_SEQUENCE;
    int rc = zq_decoder_reset_seq(m, seq, stream);
    if (rc != ZQ_OK) return rc;
    const uint32_t last = n - 1;
    if (n == 1) {  // the recorded step leaves its logits in m->logits itself
        const float* lg = nullptr;
        rc = zq_decoder_decode_next(m, seq, h_tokens[0], stream, &lg);
    } else {
        rc = zq_decoder_extend(m, seq, h_tokens, n, &last, 1, m->logits, stream);
    }
    *d_logits = m->logits;
    return rc;
}

int zq_decoder_decode_next(zq_decoder* m, uint32_t seq, uint32_t token, zq_stream stream, const float** d_logits) {
    if (!m || !d_logits || seq >= m->c.n_seq || token >= m->c.vocab) return ZQ_ERR_BAD_ARG;
    if (m->seq_lens[seq] >= m->c.ctx) return ZQ_ERR_SEQUENCE;
    cudaStream_t st = as_stream(stream);
    int rc = set_row(m, seq, token, st);
    if (rc == ZQ_OK) rc = step(m, STEP_LOGITS, 0, st);
    if (rc != ZQ_OK) return rc;
    m->seq_lens[seq] += 1;
    *d_logits = m->logits;
    return ZQ_OK;
}

int zq_decoder_decode_next_batch(zq_decoder* m, const uint32_t* h_seqs, const uint32_t* h_tokens, uint32_t n,
                                 zq_stream stream, const float** d_logits) {
    if (!m || !h_seqs || !h_tokens || !d_logits || n == 0 || n > m->c.n_seq) return ZQ_ERR_BAD_ARG;
    std::vector<uint32_t> pos(n);
    std::vector<bool> seen(m->c.n_seq, false);
    for (uint32_t r = 0; r < n; ++r) {
        const uint32_t s = h_seqs[r];
        if (s >= m->c.n_seq || seen[s] || h_tokens[r] >= m->c.vocab) return ZQ_ERR_BAD_ARG;
        if (m->seq_lens[s] >= m->c.ctx) return ZQ_ERR_SEQUENCE;
        seen[s] = true;
        pos[r] = m->seq_lens[s];
    }
    cudaStream_t st = as_stream(stream);
    ZQ_CUDA(cudaMemcpyAsync(m->d_tokens, h_tokens, n * sizeof(uint32_t), cudaMemcpyHostToDevice, st));
    ZQ_CUDA(cudaMemcpyAsync(m->d_slots, h_seqs, n * sizeof(uint32_t), cudaMemcpyHostToDevice, st));
    ZQ_CUDA(cudaMemcpyAsync(m->d_pos, pos.data(), n * sizeof(uint32_t), cudaMemcpyHostToDevice, st));
    ZQ_CUDA(cudaStreamSynchronize(st));  // the sources are host memory of the caller
    Pass P{n, false, 0, true, 0, nullptr, false, 0, 0};
    // every slot in one step is the recorded shape
    const int rc = n == m->c.n_seq ? m->graphs.run(STEP_BATCH, st, [&](cudaStream_t s) { return forward(m, P, s); })
                                   : forward(m, P, st);
    if (rc != ZQ_OK) return rc;
    for (uint32_t r = 0; r < n; ++r) m->seq_lens[h_seqs[r]] += 1;
    *d_logits = m->logits;
    return ZQ_OK;
}

int zq_decoder_decode_greedy(zq_decoder* m, uint32_t seq, uint32_t first_token, uint32_t n_steps, zq_stream stream,
                             uint32_t* h_tokens_out) {
    if (!m || !h_tokens_out || seq >= m->c.n_seq || first_token >= m->c.vocab) return ZQ_ERR_BAD_ARG;
    if (n_steps == 0) return ZQ_OK;
    if (n_steps > m->c.ctx - m->seq_lens[seq]) return ZQ_ERR_SEQUENCE;
    cudaStream_t st = as_stream(stream);
    int rc = set_row(m, seq, first_token, st);
    for (uint32_t s = 0; rc == ZQ_OK && s < n_steps; ++s) {
        rc = step(m, STEP_GREEDY, 0, st);
        if (rc == ZQ_OK) m->seq_lens[seq] += 1;
    }
    if (rc != ZQ_OK) return rc;
    ZQ_CUDA(cudaMemcpyAsync(h_tokens_out, m->d_record, n_steps * sizeof(uint32_t), cudaMemcpyDeviceToHost, st));
    ZQ_CUDA(cudaStreamSynchronize(st));
    return ZQ_OK;
}

int zq_decoder_set_trail(zq_decoder* m, float* d_trail, uint32_t rows) {
    if (!m) return ZQ_ERR_BAD_ARG;
    m->trail = d_trail;
    m->trail_rows = d_trail ? rows : 0;
    return ZQ_OK;
}

size_t zq_decoder_device_bytes(const zq_decoder* m) { return m ? m->arena.total : 0; }

}  // extern "C"
