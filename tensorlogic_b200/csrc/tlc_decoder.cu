// Runner of the config-driven decoder (tlc_decoder_* of include/tlcuda.h): dense bf16 or f32
// weights, layers described one by one.
//
// Layers over several residual streams are in tlc_decoder_streams.cu.  Layers with one residual come in
// two forms:
//   one row (a decode step, a portion of one token), three launches per layer, four with experts:
//     [norms + q, k, gate/up (or shared gate/up, router, shared gate)]
//     [q/k norm + rotation + cache append + windowed attention]
//     [router decision + gate/up of the chosen experts]            beside the attention
//     [attention output + down (+ chosen experts + shared expert) + bias, into the residual]
//   many rows (prompts, batches):
//     [norms, adding the pending expert outputs to the residual]
//     [router] [expert choice] [rows by expert]                     layers with experts
//     [q, k, gate/up and the experts' gate/up: one grouped GEMM]
//     [q/k norm + rotation + cache append] [windowed attention]
//     [attention output + down into the residual, experts' down: one grouped GEMM]
// then the final norm, the logits against the embedding table and the sampling kernels the LLaMA
// runner uses.  Token ids, positions and sampled tokens live in device memory; decode steps replay
// as CUDA graphs.
#include <algorithm>
#include <chrono>
#include <cmath>
#include <cstring>
#include <memory>

#include "tlc_decoder.h"

using namespace tlc_dense;
using namespace tlc_sample;

extern "C" int32_t tlc_model_get(tlc_model *, const char *, tlc_qtensor **);
extern "C" int32_t tlc_kvcache_create_layers(tlc_ctx *, int32_t, int32_t, int32_t, int32_t, const int32_t *, const int32_t *,
                                             tlc_kvcache **);
extern "C" int32_t tlc_kvcache_create_latent(tlc_ctx *, int32_t, int32_t, int32_t, int32_t, const int32_t *, tlc_kvcache **);
extern "C" int32_t tlc_kvcache_destroy(tlc_kvcache *);
extern "C" int32_t tlc_kvcache_layer_ptrs(tlc_kvcache *, int32_t, void **, void **);

namespace tlc_dense {

int32_t dev_alloc(tlc_decoder *D, void **p, size_t bytes) {
    cudaError_t e = cudaMalloc(p, bytes ? bytes : 16);
    if (e != cudaSuccess) {
        cudaGetLastError();
        *p = nullptr;
        return tlc_fail(TLC_ERR_ALLOCATION, "activation buffer of %zu bytes failed: %s", bytes, cudaGetErrorString(e));
    }
    D->owned.push_back(*p);
    TLC_CUDA(cudaMemsetAsync(*p, 0, bytes ? bytes : 16, D->ctx->stream));
    return TLC_OK;
}

int32_t bind_tensor(tlc_decoder *D, tlc_model *model, const std::string &name, int64_t rows, int64_t cols, tlc_qtensor **t) {
    if (int32_t rc = tlc_model_get(model, name.c_str(), t)) return rc;
    TLC_REQUIRE((*t)->n_rows == rows && (*t)->n_cols == cols, TLC_ERR_SHAPE_MISMATCH,
                "tensor '%s' is [%lld, %lld], expected [%lld, %lld]", name.c_str(), (long long)(*t)->n_rows,
                (long long)(*t)->n_cols, (long long)rows, (long long)cols);
    TLC_REQUIRE((*t)->type == D->cfg.dtype, TLC_ERR_LOAD, "tensor '%s' has type %d, the decoder runs in type %d", name.c_str(),
                (*t)->type, D->cfg.dtype);
    return TLC_OK;
}

}  // namespace tlc_dense

namespace {

// Checks the configuration of one layer.
int32_t check_layer(const tlc_decoder_layer &c, int i) {
    TLC_REQUIRE(c.mixer == TLC_MIX_WINDOW, TLC_ERR_INVALID_OPERATION, "layer %d: mixer %d needs residual streams", i, c.mixer);
    TLC_REQUIRE(c.heads > 0 && c.kv_heads > 0 && c.dim > 0 && c.heads % c.kv_heads == 0, TLC_ERR_INVALID_DIMENSION,
                "layer %d: %d heads over %d key/value heads of %d", i, c.heads, c.kv_heads, c.dim);
    TLC_REQUIRE(c.dim <= 512, TLC_ERR_INVALID_DIMENSION, "layer %d: heads of %d values (at most 512)", i, c.dim);
    TLC_REQUIRE(c.rot_dims >= 0 && c.rot_dims <= c.dim && c.rot_dims % 2 == 0 && (c.rot_dims == 0 || c.rot_base > 0),
                TLC_ERR_INVALID_DIMENSION, "layer %d: rotation of %d of %d values, base %g", i, c.rot_dims, c.dim, c.rot_base);
    TLC_REQUIRE(c.window > 0 && c.keep_first >= 0, TLC_ERR_INVALID_DIMENSION, "layer %d: window %d, kept %d", i, c.window,
                c.keep_first);
    TLC_REQUIRE(c.ff_kind == TLC_FF_NONE || c.ff_kind == TLC_FF_CLAMPED_GLU || c.ff_kind == TLC_FF_MOE, TLC_ERR_INVALID_OPERATION,
                "layer %d: unknown feed-forward %d", i, c.ff_kind);
    if (c.ff_kind == TLC_FF_CLAMPED_GLU)
        TLC_REQUIRE(c.ff > 0, TLC_ERR_INVALID_DIMENSION, "layer %d: feed-forward of width %d", i, c.ff);
    if (c.ff_kind == TLC_FF_MOE)
        TLC_REQUIRE(c.experts > 0 && c.top > 0 && c.top <= c.experts && c.expert_ff > 0 && c.shared_ff >= 0 && c.experts <= 1024,
                    TLC_ERR_INVALID_DIMENSION, "layer %d: %d of %d experts of width %d, shared %d", i, c.top, c.experts,
                    c.expert_ff, c.shared_ff);
    return TLC_OK;
}

int32_t bind(tlc_decoder *D, tlc_model *model) {
    const tlc_decoder_config &cfg = D->cfg;
    auto get = [&](const std::string &name, int64_t rows, int64_t cols, tlc_qtensor **t) { return bind_tensor(D, model, name, rows, cols, t); };
    const int64_t w = cfg.width;
    if (int32_t rc = get("embed", cfg.vocab, w, &D->embed)) return rc;
    if (int32_t rc = get("final.norm", 1, w, &D->final_norm)) return rc;
    for (int i = 0; i < cfg.n_layers; i++) {
        Layer &L = D->layers[(size_t)i];
        const tlc_decoder_layer &c = L.c;
        const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.", f = p + "mlp.";
        const int64_t qd = (int64_t)c.heads * c.dim, kd = (int64_t)c.kv_heads * c.dim;
        struct Want { tlc_qtensor **t; std::string n; int64_t r, c; };
        std::vector<Want> want = {{&L.norm1, p + "norm1", 1, w}, {&L.q, m + "q", qd, w},       {&L.qb, m + "q.b", 1, qd},
                                  {&L.qn, m + "q.norm", 1, qd},  {&L.k, m + "k", kd, w},       {&L.kb, m + "k.b", 1, kd},
                                  {&L.kn, m + "k.norm", 1, kd},  {&L.o, m + "o", w, qd},       {&L.ob, m + "o.b", 1, w}};
        if (c.ff_kind != TLC_FF_NONE) want.push_back({&L.norm2, p + "norm2", 1, w});
        if (c.ff_kind == TLC_FF_CLAMPED_GLU) {
            want.push_back({&L.gate, f + "gate", c.ff, w});
            want.push_back({&L.up, f + "up", c.ff, w});
            want.push_back({&L.down, f + "down", w, c.ff});
        }
        if (c.ff_kind == TLC_FF_MOE) {
            want.push_back({&L.router, f + "router", c.experts, w});
            L.e_gate.resize((size_t)c.experts);
            L.e_up.resize((size_t)c.experts);
            L.e_down.resize((size_t)c.experts);
            for (int e = 0; e < c.experts; e++) {
                const std::string x = f + "e" + std::to_string(e) + ".";
                want.push_back({&L.e_gate[(size_t)e], x + "gate", c.expert_ff, w});
                want.push_back({&L.e_up[(size_t)e], x + "up", c.expert_ff, w});
                want.push_back({&L.e_down[(size_t)e], x + "down", w, c.expert_ff});
            }
            if (c.shared_ff > 0) {
                want.push_back({&L.gate, f + "shared.gate", c.shared_ff, w});
                want.push_back({&L.up, f + "shared.up", c.shared_ff, w});
                want.push_back({&L.down, f + "shared.down", w, c.shared_ff});
                want.push_back({&L.sg, f + "shared.sg", 1, w});
            }
        }
        for (Want &e : want)
            if (int32_t rc = get(e.n, e.r, e.c, e.t)) return rc;
    }
    return TLC_OK;
}

// Angle factors, expert tables, activation buffers and tensor maps.
int32_t prepare(tlc_decoder *D) {
    const tlc_decoder_config &cfg = D->cfg;
    const int w = cfg.width;
    D->ldw = round8(w);
    int64_t q_max = 8, k_max = 8, rot_max = 8, attn_max = 8, act_max = 8, acte_max = 8, experts_max = 1;
    for (Layer &L : D->layers) {
        const tlc_decoder_layer &c = L.c;
        q_max = std::max<int64_t>(q_max, round8(c.heads * c.dim));
        k_max = std::max<int64_t>(k_max, round8(c.kv_heads * c.dim));
        rot_max = std::max<int64_t>(rot_max, (int64_t)c.heads * round8(c.dim));
        attn_max = std::max<int64_t>(attn_max, round8(c.heads * c.dim));
        act_max = std::max<int64_t>(act_max, round8(L.ff_width()));
        ExpertParams ep{};
        OutParams op{};
        op.n = ep.k = w;
        op.seg[op.n_seg++].k = c.heads * c.dim;
        if (L.ff_width()) op.seg[op.n_seg++].k = L.ff_width();
        if (c.ff_kind == TLC_FF_MOE) {
            acte_max = std::max<int64_t>(acte_max, (int64_t)round8(c.expert_ff));
            experts_max = std::max<int64_t>(experts_max, c.experts);
            D->top_max = std::max(D->top_max, c.top);
            ep.experts = c.experts;
            ep.top = op.top = c.top;
            ep.ff = op.expert_k = c.expert_ff;
        }
        const bool fits = cfg.dtype == TLC_TYPE_F32 ? layer_gemv_fits<float>(D->ctx, ep, op) : layer_gemv_fits<bf16>(D->ctx, ep, op);
        if (!gemv_fits(w) || !fits) D->one_row_ok = false;
        if (c.rot_dims > 0) {
            std::vector<float> fr((size_t)c.rot_dims / 2);
            for (size_t i = 0; i < fr.size(); i++) fr[i] = (float)std::pow(c.rot_base, -2.0 * (double)i / (double)c.rot_dims);
            if (int32_t rc = upload(D, &L.freq, fr.data(), fr.size() * 4)) return rc;
        }
        if (c.ff_kind == TLC_FF_MOE) {
            std::vector<const void *> t((size_t)c.experts);
            struct { const std::vector<tlc_qtensor *> &src; const void ***dst; } tabs[] = {
                {L.e_gate, &L.gate_tab}, {L.e_up, &L.up_tab}, {L.e_down, &L.down_tab}};
            for (auto &tb : tabs) {
                for (size_t e = 0; e < t.size(); e++) t[e] = tb.src[e]->data;
                if (int32_t rc = upload(D, tb.dst, t.data(), t.size() * sizeof(void *))) return rc;
            }
        }
    }
    // buffers of the form with one residual
    const size_t one = cfg.streams ? 0 : 1, R = (size_t)D->rows, es = D->elem, pairs = R * (size_t)std::max(D->top_max, 1);
    D->ld_router = (int)experts_max + 1;
    struct { void **p; size_t bytes; } bufs[] = {
        {(void **)&D->x, one * R * w * 4},
        {(void **)&D->h_row, one * (size_t)D->ldw * 4},
        {(void **)&D->h1, one * R * D->ldw * es},
        {(void **)&D->h2, one * R * D->ldw * es},
        {(void **)&D->q_raw, one * R * q_max * es},
        {(void **)&D->k_raw, one * R * k_max * es},
        {(void **)&D->q_rot, one * R * rot_max * es},
        {(void **)&D->attn, one * R * attn_max * es},
        {(void **)&D->act, one * R * act_max * es},
        {(void **)&D->router_out, R * D->ld_router * 4},
        {(void **)&D->chosen, one * pairs * 4},
        {(void **)&D->rank, one * pairs * 4},
        {(void **)&D->place, one * pairs * 4},
        {(void **)&D->weight, one * pairs * 4},
        {(void **)&D->scale, one * pairs * 4},
        {(void **)&D->count, (size_t)experts_max * 4},
        {(void **)&D->off, (size_t)(experts_max + 1) * 4},
        {(void **)&D->hp, D->top_max ? pairs * D->ldw * es : 0},
        {(void **)&D->act_e, D->top_max ? pairs * acte_max * es : 0},
        {(void **)&D->y, D->top_max ? pairs * D->ldw * es : 0},
        {(void **)&D->hf, (size_t)D->logit_rows * D->ldw * es},
        {(void **)&D->logits, (size_t)D->logit_rows * cfg.vocab * 4},
        {(void **)&D->row_ids, R * 4},
        {(void **)&D->row_pos, R * 4},
        {(void **)&D->row_slot, R * 4},
        {(void **)&D->want, (size_t)D->logit_rows * 4},
        {(void **)&D->ids, kMaxSeqs * 4},
        {(void **)&D->positions, kMaxSeqs * 4},
        {(void **)&D->next_ids, kMaxSeqs * 4},
    };
    for (auto &b : bufs)
        if (int32_t rc = dev_alloc(D, b.p, b.bytes)) return rc;
    int iota[kMaxSeqs];
    for (int i = 0; i < kMaxSeqs; i++) iota[i] = i;
    if (int32_t rc = upload(D, &D->slots, iota, sizeof iota)) return rc;
    TLC_CUDA(cudaMallocHost(&D->host_rows, (3 * R + (size_t)D->logit_rows) * 4));
    TLC_CUDA(cudaMallocHost(&D->host_next, 64 * 4));
    TLC_CUDA(cudaMallocHost(&D->host_ids, 64 * 4));

    Maps maps;
    if (cfg.streams)
        if (int32_t rc = prepare_streams(D, maps)) return rc;
    if (cfg.dtype != TLC_TYPE_BF16) return TLC_OK;
    auto add = [&](const void *base, int64_t rows, int64_t cols, int64_t pitch) { return maps.add(base, rows, cols, pitch); };
    auto weight = [&](const tlc_qtensor *t) { return maps.weight(t); };
    if (one) {
        D->a_h1 = add(D->h1, (int64_t)R, w, D->ldw);
        D->a_h2 = add(D->h2, (int64_t)R, w, D->ldw);
    }
    if (D->top_max) D->a_hp = add(D->hp, (int64_t)pairs, w, D->ldw);
    D->a_hf = add(D->hf, D->logit_rows, w, D->ldw);
    D->m_embed = weight(D->embed);
    for (Layer &L : D->layers) {
        const tlc_decoder_layer &c = L.c;
        const int qd = c.heads * c.dim;
        L.a_attn = add(D->attn, (int64_t)R, qd, round8(qd));
        L.m_q = weight(L.q);
        L.m_k = weight(L.k);
        L.m_o = weight(L.o);
        if (L.gate) {
            L.a_act = add(D->act, (int64_t)R, L.ff_width(), round8(L.ff_width()));
            L.m_gate = weight(L.gate);
            L.m_up = weight(L.up);
            L.m_down = weight(L.down);
        }
        if (L.router) {
            L.m_router = weight(L.router);
            if (L.sg) L.m_sg = weight(L.sg);
            L.a_acte = add(D->act_e, (int64_t)pairs, c.expert_ff, round8(c.expert_ff));
            struct { const std::vector<tlc_qtensor *> &src; int *first; } fam[] = {
                {L.e_gate, &L.m_egate}, {L.e_up, &L.m_eup}, {L.e_down, &L.m_edown}};
            for (auto &f : fam) {
                *f.first = (int)maps.maps.size();
                for (const tlc_qtensor *t : f.src) weight(t);
            }
        }
    }
    if (maps.bad) return maps.bad;
    return upload(D, &D->maps, maps.maps.data(), maps.maps.size() * sizeof(CUtensorMap));
}

template <typename T>
int32_t layer_attention(tlc_decoder *D, Layer &L, int l, const Pass &ps, bool one_row) {
    const tlc_decoder_layer &c = L.c;
    void *kc = nullptr, *vc = nullptr;
    tlc_kvcache_layer_ptrs(D->cache, l, &kc, &vc);
    WindowAttn a{};
    a.ldq = round8(c.heads * c.dim);
    a.ldk = round8(c.kv_heads * c.dim);
    a.qn = L.qn->data;
    a.kn = L.kn->data;
    a.freq = L.freq;
    a.rot = c.rot_dims;
    a.eps = D->cfg.norm_eps;
    a.kc = kc;
    a.vc = vc;
    a.out = D->attn;
    a.ldo = round8(c.heads * c.dim);
    a.H = c.heads;
    a.G = c.kv_heads;
    a.D = c.dim;
    a.Dp = round8(c.dim);
    a.window = c.window;
    a.keep = c.keep_first;
    a.scale = c.scale;
    a.pos = ps.pos;
    a.slot = ps.slot;
    a.max_seq = D->cfg.max_seq;
    a.m = ps.m;
    a.pos0 = ps.pos0;
    a.status = D->ctx->dev_status;
    const bool tensor = sizeof(T) == 2 && window_tensor_cores(c.dim);
    if (tensor && (ps.decode || one_row)) {
        a.q = D->q_raw;
        a.k_raw = D->k_raw;
        return launch_window_decode(D->ctx, a);
    }
    RotParams r{};
    r.q = D->q_raw;
    r.k = D->k_raw;
    r.ldq = a.ldq;
    r.ldk = a.ldk;
    r.qn = a.qn;
    r.kn = a.kn;
    r.freq = a.freq;
    r.H = a.H;
    r.G = a.G;
    r.D = a.D;
    r.Dp = a.Dp;
    r.rot = a.rot;
    r.eps = a.eps;
    r.pos = a.pos;
    r.slot = a.slot;
    r.max_seq = a.max_seq;
    r.q_out = D->q_rot;
    r.kc = kc;
    r.vc = vc;
    r.status = a.status;
    if (int32_t rc = launch_qk_rotate<T>(D->ctx, r, ps.m)) return rc;
    a.q = D->q_rot;
    if (tensor) return launch_window_prefill(D->ctx, a, ps.seq);
    return launch_window_rows<T>(D->ctx, a);
}

// One row: the streaming kernels.
template <typename T>
int32_t layers_one_row(tlc_decoder *D, const Pass &ps) {
    tlc_ctx *ctx = D->ctx;
    const int w = D->cfg.width, es = (int)sizeof(T);
    for (int l = 0; l < (int)D->runs.size(); l++) {
        Layer &L = D->layers[(size_t)D->runs[(size_t)l]];
        const tlc_decoder_layer &c = L.c;
        const bool moe = c.ff_kind == TLC_FF_MOE;
        GemvParams g{};
        g.k = w;
        g.pitch = (int)(L.q->row_pitch / es);
        g.x = D->x;
        g.norm_w[0] = L.norm1->data;
        g.norm_w[1] = L.norm2 ? L.norm2->data : L.norm1->data;
        g.eps = D->cfg.norm_eps;
        auto seg = [&](const tlc_qtensor *t, const tlc_qtensor *t2, const tlc_qtensor *bias, void *out, int epi, int input) {
            GemvSeg &s = g.seg[g.n_seg++];
            s.w = t->data;
            s.w2 = t2 ? t2->data : nullptr;
            s.bias = bias ? bias->data : nullptr;
            s.out = out;
            s.n = (int)t->n_rows;
            s.epi = epi;
            s.input = input;
            s.limit = c.limit;
        };
        seg(L.q, nullptr, L.qb, D->q_raw, EPI_STORE, 0);
        seg(L.k, nullptr, L.kb, D->k_raw, EPI_STORE, 0);
        if (L.gate) seg(L.gate, L.up, nullptr, D->act, moe ? EPI_SILU_MUL : EPI_CLAMPED_GLU, 1);
        if (moe) {
            seg(L.router, nullptr, nullptr, D->router_out, EPI_STORE_F32, 1);
            if (L.sg) seg(L.sg, nullptr, nullptr, D->router_out + c.experts, EPI_STORE_F32, 1);
            g.h_out = D->h_row;
        }
        if (int32_t rc = launch_gemv<T>(ctx, g)) return rc;
        if (int32_t rc = layer_attention<T>(D, L, l, ps, true)) return rc;
        if (moe) {
            ExpertParams e{};
            e.h = D->h_row;
            e.logits = D->router_out;
            e.gate = L.gate_tab;
            e.up = L.up_tab;
            e.act = D->act_e;
            e.chosen = D->chosen;
            e.weight = D->weight;
            e.experts = c.experts;
            e.top = c.top;
            e.k = w;
            e.pitch = g.pitch;
            e.ff = c.expert_ff;
            e.act_pitch = round8(c.expert_ff);
            if (int32_t rc = launch_expert_gemv<T>(ctx, e)) return rc;
        }
        OutParams o{};
        o.seg[o.n_seg++] = {L.o->data, D->attn, (int)L.o->n_cols, (int)(L.o->row_pitch / es), 0, 1, nullptr};
        if (L.down)
            o.seg[o.n_seg++] = {L.down->data, D->act, (int)L.down->n_cols, (int)(L.down->row_pitch / es), 0, 1,
                                L.sg ? D->router_out + c.experts : nullptr};
        if (moe) {
            o.down = L.down_tab;
            o.chosen = D->chosen;
            o.expert_in = D->act_e;
            o.top = c.top;
            o.expert_k = c.expert_ff;
            o.expert_pitch = (int)(L.e_down[0]->row_pitch / es);
            o.expert_in_pitch = round8(c.expert_ff);
        }
        o.bias = L.ob->data;
        o.x = D->x;
        o.n = w;
        if (int32_t rc = launch_out_gemv<T>(ctx, o)) return rc;
    }
    return TLC_OK;
}

// Many rows.  On return `pending` names the layer whose expert outputs are not in x yet, or -1.
template <typename T>
int32_t layers_many_rows(tlc_decoder *D, const Pass &ps, int *pending) {
    tlc_ctx *ctx = D->ctx;
    const int w = D->cfg.width, m = ps.m;
    *pending = -1;
    for (int l = 0; l < (int)D->runs.size(); l++) {
        Layer &L = D->layers[(size_t)D->runs[(size_t)l]];
        const tlc_decoder_layer &c = L.c;
        const bool moe = c.ff_kind == TLC_FF_MOE;
        const int qd = c.heads * c.dim, kd = c.kv_heads * c.dim, ff = L.ff_width();
        NormParams n{};
        n.x = D->x;
        n.m = m;
        n.d = w;
        n.w[0] = L.norm1->data;
        n.out[0] = D->h1;
        n.w[1] = L.norm2 ? L.norm2->data : nullptr;
        n.out[1] = D->h2;
        n.ldo = D->ldw;
        n.eps = D->cfg.norm_eps;
        if (*pending >= 0) {
            n.y = D->y;
            n.place = D->place;
            n.top = D->layers[(size_t)*pending].c.top;
            n.y_pitch = D->ldw;
            *pending = -1;
        }
        if (moe) {
            n.zero = D->count;
            n.n_zero = c.experts;
        }
        if (int32_t rc = launch_norm<T>(ctx, n)) return rc;
        if (moe) {
            Gemm<T> r(D, m);
            r.operand(r.add(c.experts, EPI_STORE_F32, D->router_out, D->ld_router), 0, D->a_h2, D->h2, D->ldw, L.m_router, L.router);
            if (L.sg)
                r.operand(r.add(1, EPI_STORE_F32, D->router_out + c.experts, D->ld_router), 0, D->a_h2, D->h2, D->ldw, L.m_sg, L.sg);
            if (int32_t rc = r.launch()) return rc;
            RouteParams rt{};
            rt.logits = D->router_out;
            rt.ld = D->ld_router;
            rt.experts = c.experts;
            rt.top = c.top;
            rt.m = m;
            rt.chosen = D->chosen;
            rt.rank = D->rank;
            rt.count = D->count;
            rt.weight = D->weight;
            if (int32_t rc = launch_route(ctx, rt)) return rc;
            PermuteParams pm{};
            pm.h = D->h2;
            pm.m = m;
            pm.d = w;
            pm.ldh = D->ldw;
            pm.top = c.top;
            pm.experts = c.experts;
            pm.chosen = D->chosen;
            pm.rank = D->rank;
            pm.count = D->count;
            pm.weight = D->weight;
            pm.off = D->off;
            pm.place = D->place;
            pm.hp = D->hp;
            pm.scale = D->scale;
            if (int32_t rc = launch_permute<T>(ctx, pm)) return rc;
        }
        auto family = [&](GemmGroup &g, const void *const *tab, const void *const *tab2) {
            g.experts = c.experts;
            g.map_stride = 1;
            g.off = D->off;
            g.in_rows_per_token = c.top;
            g.b_tab = tab;
            g.b2_tab = tab2;
        };
        {
            Gemm<T> a(D, m);
            GemmGroup &gq = a.add(qd, EPI_STORE, D->q_raw, round8(qd));
            a.operand(gq, 0, D->a_h1, D->h1, D->ldw, L.m_q, L.q);
            gq.bias = L.qb->data;
            if (L.gate) {
                GemmGroup &g = a.add(ff, moe ? EPI_SILU_MUL : EPI_CLAMPED_GLU, D->act, round8(ff));
                a.operand(g, 0, D->a_h2, D->h2, D->ldw, L.m_gate, L.gate);
                g.b2_map = L.m_up;
                g.b2 = L.up->data;
                g.limit = c.limit;
                if (L.sg) {
                    g.out_scale = D->router_out + c.experts;
                    g.out_scale_stride = D->ld_router;
                }
            }
            if (moe) {
                GemmGroup &g = a.add(c.expert_ff, EPI_SILU_MUL, D->act_e, round8(c.expert_ff));
                a.operand(g, 0, D->a_hp, D->hp, D->ldw, L.m_egate, L.e_gate[0]);
                g.b2_map = L.m_eup;
                g.in_scale = D->scale;
                family(g, L.gate_tab, L.up_tab);
            }
            GemmGroup &gk = a.add(kd, EPI_STORE, D->k_raw, round8(kd));
            a.operand(gk, 0, D->a_h1, D->h1, D->ldw, L.m_k, L.k);
            gk.bias = L.kb->data;
            if (int32_t rc = a.launch()) return rc;
        }
        if (int32_t rc = layer_attention<T>(D, L, l, ps, false)) return rc;
        {
            Gemm<T> b(D, m);
            GemmGroup &g = b.add(w, EPI_ADD_F32, D->x, w);
            b.operand(g, 0, L.a_attn, D->attn, round8(qd), L.m_o, L.o);
            if (L.down) b.operand(g, 1, L.a_act, D->act, round8(ff), L.m_down, L.down);
            g.bias = L.ob->data;
            if (moe) {
                GemmGroup &e = b.add(w, EPI_STORE, D->y, D->ldw);
                b.operand(e, 0, L.a_acte, D->act_e, round8(c.expert_ff), L.m_edown, L.e_down[0]);
                family(e, L.down_tab, nullptr);
                *pending = D->runs[(size_t)l];
            }
            if (int32_t rc = b.launch()) return rc;
        }
    }
    return TLC_OK;
}

template <typename T>
int32_t forward_t(tlc_decoder *D, const Pass &ps) {
    tlc_ctx *ctx = D->ctx;
    const int w = D->cfg.width;
    if (int32_t rc = launch_embed<T>(ctx, D->embed, ps.ids, ps.m, D->x)) return rc;
    int pending = -1;
    if (ps.m == 1 && D->one_row_ok) {
        if (int32_t rc = layers_one_row<T>(D, ps)) return rc;
    } else {
        if (int32_t rc = layers_many_rows<T>(D, ps, &pending)) return rc;
    }
    const int n = ps.want || ps.n_want ? ps.n_want : ps.m;
    if (n == 0) return TLC_OK;
    const bool single = n == 1 && gemv_fits(w);
    // the one-row kernel takes a residual row that starts on a 16-byte boundary
    const bool fused = single && pending < 0 && (ps.m == 1 || (ps.want_single >= 0 && w % 4 == 0));
    if (!fused) {
        NormParams np{};
        np.x = D->x;
        np.m = n;
        np.d = w;
        np.rows = ps.want;
        np.w[0] = D->final_norm->data;
        np.out[0] = D->hf;
        np.ldo = D->ldw;
        np.eps = D->cfg.norm_eps;
        if (pending >= 0) {
            np.y = D->y;
            np.place = D->place;
            np.top = D->layers[(size_t)pending].c.top;
            np.y_pitch = D->ldw;
        }
        if (int32_t rc = launch_norm<T>(ctx, np)) return rc;
    }
    if (single) {
        GemvParams g{};
        g.k = w;
        g.pitch = (int)(D->embed->row_pitch / sizeof(T));
        g.x = D->x + (size_t)(ps.m == 1 ? 0 : ps.want_single < 0 ? 0 : ps.want_single) * w;
        g.xn = fused ? nullptr : D->hf;
        g.norm_w[0] = g.norm_w[1] = D->final_norm->data;
        g.eps = D->cfg.norm_eps;
        g.n_seg = 1;
        g.seg[0].w = D->embed->data;
        g.seg[0].out = D->logits;
        g.seg[0].n = D->cfg.vocab;
        g.seg[0].epi = EPI_STORE_F32;
        return launch_gemv<T>(ctx, g);
    }
    Gemm<T> lm(D, n);
    lm.operand(lm.add(D->cfg.vocab, EPI_STORE_F32, D->logits, D->cfg.vocab), 0, D->a_hf, D->hf, D->ldw, D->m_embed, D->embed);
    return lm.launch();
}

int32_t forward(tlc_decoder *D, const Pass &ps) {
    if (D->cfg.streams) return forward_streams(D, ps);
    return D->cfg.dtype == TLC_TYPE_F32 ? forward_t<float>(D, ps) : forward_t<bf16>(D, ps);
}

int32_t sample(tlc_decoder *D, const float *logits, int rows, int fixed_pos, int seq0, int *next, int *ids, int *positions, bool advance) {
    tlc_ctx *ctx = D->ctx;
    cudaError_t le = D->temperature > 0.0001f
                         ? tlc_launch_pdl(ctx, sample_advance_kernel<float>, dim3(rows), dim3(1024), 0, logits, D->cfg.vocab, 1,
                                          rows, D->temperature, D->seed, (const float *)nullptr, fixed_pos, seq0, next, ids, positions,
                                          advance ? 1 : 0, D->report)
                         : tlc_launch_pdl(ctx, argmax_advance_kernel<float>, dim3(rows), dim3(1024), 0, logits, D->cfg.vocab, 1,
                                          rows, next, ids, positions, advance ? 1 : 0, D->report);
    if (le != cudaSuccess) {
        cudaGetLastError();
        return tlc_fail(TLC_ERR_CUDA, "sampling launch failed: %s", cudaGetErrorString(le));
    }
    TLC_CHECK_LAUNCH(ctx);
    return TLC_OK;
}

int32_t decode_step(tlc_decoder *D, int batch, bool advance) {
    Pass ps{};
    ps.m = batch;
    ps.ids = D->ids_src ? D->ids_src : D->ids;
    ps.pos = D->positions;
    ps.slot = D->slots;
    ps.decode = true;
    if (int32_t rc = forward(D, ps)) return rc;
    return sample(D, D->logits, batch, -1, 0, D->next_ids, D->ids, D->positions, advance);
}

int32_t check_ids(const tlc_decoder *D, const int32_t *ids, int n) {
    for (int i = 0; i < n; i++)
        TLC_REQUIRE(ids[i] >= 0 && ids[i] < D->cfg.vocab, TLC_ERR_INDEX, "Index out of bounds: index %d, size %d", ids[i],
                    D->cfg.vocab);
    return TLC_OK;
}

// A decode step at position p writes cache row p.
int32_t reserve_positions(tlc_decoder *D, int batch, int steps) {
    int hi = 0;
    for (int i = 0; i < batch; i++) hi = D->pos_hi[(size_t)i] > hi ? D->pos_hi[(size_t)i] : hi;
    TLC_REQUIRE((int64_t)hi + steps <= D->cfg.max_seq, TLC_ERR_INDEX, "Index out of bounds: index %d, size %d", hi + steps,
                D->cfg.max_seq);
    for (int i = 0; i < batch; i++) D->pos_hi[(size_t)i] += steps;
    return TLC_OK;
}

// The step as a graph under `key`, captured on first use (after one run that warms the kernels'
// attributes and does not advance).
int32_t step_graph(tlc_decoder *D, int batch, int key) {
    tlc_ctx *ctx = D->ctx;
    if (D->graph.count(key)) return TLC_OK;
    const HostReport keep_report = D->report;
    const int *keep_src = D->ids_src;
    D->report = HostReport{};
    D->ids_src = nullptr;
    // the warm-up run writes the cache row of the pending position, which the real step writes again
    int32_t rc = decode_step(D, batch, false);
    D->report = keep_report;
    D->ids_src = keep_src;
    if (rc) return rc;
    TLC_CUDA(cudaStreamSynchronize(ctx->stream));
    const uint64_t before = ctx->launches;
    TLC_CUDA(cudaStreamBeginCapture(ctx->stream, cudaStreamCaptureModeThreadLocal));
    rc = decode_step(D, batch, true);
    cudaGraph_t g = nullptr;
    cudaError_t e = cudaStreamEndCapture(ctx->stream, &g);
    D->launches = (int)(ctx->launches - before);
    ctx->launches = before;
    if (rc) {
        if (g) cudaGraphDestroy(g);
        return rc;
    }
    if (e != cudaSuccess) return tlc_fail(TLC_ERR_CUDA, "graph capture failed: %s", cudaGetErrorString(e));
    cudaGraphExec_t ge = nullptr;
    e = cudaGraphInstantiate(&ge, g, 0);
    cudaGraphDestroy(g);
    if (e != cudaSuccess) return tlc_fail(TLC_ERR_CUDA, "graph instantiate failed: %s", cudaGetErrorString(e));
    D->graph[key] = ge;
    return TLC_OK;
}

void drop_graphs(tlc_decoder *D) {
    for (auto &g : D->graph)
        if (g.second) cudaGraphExecDestroy(g.second);
    D->graph.clear();
}

}  // namespace

extern "C" int32_t tlc_decoder_destroy(tlc_decoder *D) {
    if (!D) return TLC_OK;
    cudaSetDevice(D->ctx->device);
    cudaStreamSynchronize(D->ctx->stream);
    drop_graphs(D);
    tlc_kvcache_destroy(D->cache);
    for (void *p : D->owned) cudaFree(p);
    cudaFreeHost(D->host_rows);
    cudaFreeHost(D->host_next);
    cudaFreeHost(D->host_ids);
    delete D;
    return TLC_OK;
}

extern "C" int32_t tlc_decoder_create(tlc_ctx *ctx, tlc_model *model, const tlc_decoder_config *cfg, tlc_decoder **out) {
    if (int32_t rc = tlc_enter(ctx)) return rc;
    TLC_REQUIRE(model && cfg && out && cfg->layers, TLC_ERR_INVALID_OPERATION, "decoder_create: null pointer");
    *out = nullptr;
    const tlc_decoder_config &c = *cfg;
    TLC_REQUIRE(c.dtype == TLC_TYPE_BF16 || c.dtype == TLC_TYPE_F32, TLC_ERR_INVALID_OPERATION, "decoder_create: type %d (bf16 or f32)",
                c.dtype);
    TLC_REQUIRE(c.n_layers > 0 && c.width > 0 && c.vocab > 0 && c.max_seq > 0 && c.max_batch > 0 && c.max_batch <= kMaxSeqs &&
                    c.max_logit_rows >= 0,
                TLC_ERR_INVALID_DIMENSION, "decoder_create: bad configuration");
    TLC_REQUIRE(c.width <= 50 * 1024, TLC_ERR_INVALID_DIMENSION, "decoder_create: width %d (at most 51200)", c.width);
    std::unique_ptr<tlc_decoder, int32_t (*)(tlc_decoder *)> D(new tlc_decoder(), tlc_decoder_destroy);
    D->ctx = ctx;
    D->cfg = c;
    D->elem = c.dtype == TLC_TYPE_F32 ? 4 : 2;
    D->rows = std::max(std::max(c.max_prefill, c.max_batch), 16);
    D->logit_rows = std::max(std::min(c.max_logit_rows, D->rows), c.max_batch) + 1;  // and the row that is sampled
    D->pos_hi.assign(kMaxSeqs, 0);
    TLC_REQUIRE(c.streams >= 0 && c.streams <= kMaxStreams, TLC_ERR_INVALID_DIMENSION, "decoder_create: %d residual streams (at most %d)",
                c.streams, kMaxStreams);
    TLC_REQUIRE(c.logit_softcap >= 0.f && (c.streams || c.logit_softcap == 0.f), TLC_ERR_INVALID_OPERATION,
                "decoder_create: logit softcap %g", (double)c.logit_softcap);
    TLC_REQUIRE(c.n_runs >= 0 && (c.n_runs == 0 || c.runs), TLC_ERR_INVALID_OPERATION, "decoder_create: %d runs", c.n_runs);
    for (int r = 0; r < (c.n_runs ? c.n_runs : c.n_layers); r++) {
        const int l = c.n_runs ? c.runs[r] : r;
        TLC_REQUIRE(l >= 0 && l < c.n_layers, TLC_ERR_INDEX, "Index out of bounds: index %d, size %d", l, c.n_layers);
        D->runs.push_back(l);
    }
    for (int i = 0; i < c.n_layers; i++)
        if (int32_t rc = c.streams ? check_stream_layer(c.layers[i], i) : check_layer(c.layers[i], i)) return rc;
    std::vector<int32_t> heads, dims, latents;
    if (c.streams) {
        D->st.layers.resize((size_t)c.n_layers);
        for (int i = 0; i < c.n_layers; i++) {
            StreamLayer &L = D->st.layers[(size_t)i];
            L.c = c.layers[i];
            L.kp = round8(L.c.kv_rank);
            L.row = L.kp + round8(L.c.rot_dims);
        }
        for (int l : D->runs) latents.push_back(D->st.layers[(size_t)l].row);
    } else {
        D->layers.resize((size_t)c.n_layers);
        for (int i = 0; i < c.n_layers; i++) D->layers[(size_t)i].c = c.layers[i];
        for (int l : D->runs) {
            heads.push_back(c.layers[l].kv_heads);
            dims.push_back(c.layers[l].dim);
        }
    }
    D->cfg.layers = nullptr;  // the caller's arrays
    D->cfg.runs = nullptr;
    const int runs = (int)D->runs.size();
    if (int32_t rc = c.streams ? bind_streams(D.get(), model) : bind(D.get(), model)) return rc;
    if (int32_t rc = c.streams ? tlc_kvcache_create_latent(ctx, c.dtype, runs, c.max_batch, c.max_seq, latents.data(), &D->cache)
                               : tlc_kvcache_create_layers(ctx, c.dtype, runs, c.max_batch, c.max_seq, heads.data(), dims.data(), &D->cache))
        return rc;
    if (int32_t rc = prepare(D.get())) return rc;
    TLC_CUDA(cudaFuncSetAttribute(argmax_advance_kernel<float>, cudaFuncAttributePreferredSharedMemoryCarveout,
                                  cudaSharedmemCarveoutMaxShared));
    TLC_CUDA(cudaStreamSynchronize(ctx->stream));
    *out = D.release();
    return TLC_OK;
}

extern "C" int32_t tlc_decoder_prefill(tlc_decoder *D, int32_t seq, const int32_t *ids_host, int32_t n, int32_t pos0,
                                       const int32_t *want, int32_t n_want, float *logits_host, int32_t *next_id_host) {
    TLC_REQUIRE(D && ids_host && (n_want == 0 || (want && logits_host)), TLC_ERR_INVALID_OPERATION, "decoder_prefill: null pointer");
    tlc_ctx *ctx = D->ctx;
    if (int32_t rc = tlc_enter(ctx)) return rc;
    tlc_perf_scope perf(ctx, "decoder_prefill(tokens=%d)", n);
    TLC_REQUIRE(seq >= 0 && seq < D->cfg.max_batch, TLC_ERR_INDEX, "Index out of bounds: index %d, size %d", seq, D->cfg.max_batch);
    TLC_REQUIRE(n >= 1 && n_want >= 0 && n_want <= n, TLC_ERR_SHAPE_MISMATCH, "prefill of %d tokens, %d wanted", n, n_want);
    TLC_REQUIRE(pos0 >= 0 && n <= D->cfg.max_seq - pos0, TLC_ERR_INDEX, "Index out of bounds: index %lld, size %d",
                (long long)pos0 + n, D->cfg.max_seq);
    TLC_REQUIRE(pos0 <= D->pos_hi[(size_t)seq], TLC_ERR_INDEX, "sequence %d ends at position %d: no portion can start at %d", seq,
                D->pos_hi[(size_t)seq], pos0);
    for (int i = 0; i < n_want; i++)
        TLC_REQUIRE(want[i] >= 0 && want[i] < n && (i == 0 || want[i] > want[i - 1]), TLC_ERR_INDEX,
                    "wanted places must ascend within the %d tokens", n);
    if (int32_t rc = check_ids(D, ids_host, n)) return rc;
    const size_t R = (size_t)D->rows;
    int *h_ids = D->host_rows, *h_pos = h_ids + R, *h_slot = h_pos + R, *h_want = h_slot + R;
    int done_want = 0;
    for (int at = 0; at < n;) {
        // a stretch: at most `rows` rows and one logit row less than there is room for
        int len = std::min(n - at, D->rows), w = 0;
        while (done_want + w < n_want && want[done_want + w] < at + len) {
            if (w == D->logit_rows - 1) {
                len = want[done_want + w] - at;
                break;
            }
            w++;
        }
        const bool last = at + len == n;
        const bool draw = last && next_id_host;
        for (int i = 0; i < len; i++) {
            h_ids[i] = ids_host[at + i];
            h_pos[i] = pos0 + at + i;
            h_slot[i] = seq;
        }
        for (int i = 0; i < w; i++) h_want[i] = want[done_want + i] - at;
        int rows = w;
        if (draw && (w == 0 || h_want[w - 1] != len - 1)) h_want[rows++] = len - 1;
        TLC_CUDA(cudaMemcpyAsync(D->row_ids, h_ids, (size_t)len * 4, cudaMemcpyHostToDevice, ctx->stream));
        TLC_CUDA(cudaMemcpyAsync(D->row_pos, h_pos, (size_t)len * 4, cudaMemcpyHostToDevice, ctx->stream));
        TLC_CUDA(cudaMemcpyAsync(D->row_slot, h_slot, (size_t)len * 4, cudaMemcpyHostToDevice, ctx->stream));
        if (rows) TLC_CUDA(cudaMemcpyAsync(D->want, h_want, (size_t)rows * 4, cudaMemcpyHostToDevice, ctx->stream));
        Pass ps{};
        ps.m = len;
        ps.ids = D->row_ids;
        ps.pos = D->row_pos;
        ps.slot = D->row_slot;
        ps.seq = seq;
        ps.pos0 = pos0 + at;
        ps.want = D->want;
        ps.n_want = rows;
        ps.want_single = rows == 1 ? h_want[0] : -1;
        if (int32_t rc = forward(D, ps)) return rc;
        if (w)
            TLC_CUDA(cudaMemcpyAsync(logits_host + (size_t)done_want * D->cfg.vocab, D->logits, (size_t)w * D->cfg.vocab * 4,
                                     cudaMemcpyDeviceToHost, ctx->stream));
        if (draw) {
            if (int32_t rc = sample(D, D->logits + (size_t)(rows - 1) * D->cfg.vocab, 1, pos0 + n - 1, seq, D->next_ids + seq, nullptr,
                                    nullptr, false))
                return rc;
            TLC_CUDA(cudaMemcpyAsync(D->ids + seq, D->next_ids + seq, 4, cudaMemcpyDeviceToDevice, ctx->stream));
            TLC_CUDA(cudaMemcpyAsync(D->host_next, D->next_ids + seq, 4, cudaMemcpyDeviceToHost, ctx->stream));
        }
        done_want += w;
        at += len;
        if (last) {
            // the sequence continues behind the portion
            D->host_next[32] = pos0 + n;
            TLC_CUDA(cudaMemcpyAsync(D->positions + seq, &D->host_next[32], 4, cudaMemcpyHostToDevice, ctx->stream));
        }
        if (int32_t rc = tlc_synchronize(ctx)) return rc;  // the pinned rows are filled again
    }
    D->pos_hi[(size_t)seq] = pos0 + n;
    if (next_id_host) *next_id_host = D->host_next[0];
    return TLC_OK;
}

extern "C" int32_t tlc_decoder_release(tlc_decoder *D, int32_t seq) {
    TLC_REQUIRE(D, TLC_ERR_INVALID_OPERATION, "decoder_release: null handle");
    TLC_REQUIRE(seq >= 0 && seq < D->cfg.max_batch, TLC_ERR_INDEX, "Index out of bounds: index %d, size %d", seq, D->cfg.max_batch);
    if (int32_t rc = tlc_enter(D->ctx)) return rc;
    TLC_CUDA(cudaMemsetAsync(D->positions + seq, 0, 4, D->ctx->stream));
    TLC_CUDA(cudaMemsetAsync(D->ids + seq, 0, 4, D->ctx->stream));
    D->pos_hi[(size_t)seq] = 0;
    return TLC_OK;
}

extern "C" int32_t tlc_decoder_set_state(tlc_decoder *D, int32_t batch, const int32_t *ids_host, const int32_t *positions_host) {
    TLC_REQUIRE(D && ids_host && positions_host, TLC_ERR_INVALID_OPERATION, "decoder_set_state: null pointer");
    if (int32_t rc = tlc_enter(D->ctx)) return rc;
    TLC_REQUIRE(batch >= 1 && batch <= D->cfg.max_batch, TLC_ERR_SHAPE_MISMATCH, "batch %d (max %d)", batch, D->cfg.max_batch);
    if (int32_t rc = check_ids(D, ids_host, batch)) return rc;
    for (int i = 0; i < batch; i++)
        TLC_REQUIRE(positions_host[i] >= 0 && positions_host[i] < D->cfg.max_seq, TLC_ERR_INDEX, "Index out of bounds: index %d, size %d",
                    positions_host[i], D->cfg.max_seq);
    TLC_CUDA(cudaStreamSynchronize(D->ctx->stream));  // earlier steps may still read ids / positions
    TLC_CUDA(cudaMemcpy(D->ids, ids_host, (size_t)batch * 4, cudaMemcpyHostToDevice));
    TLC_CUDA(cudaMemcpy(D->positions, positions_host, (size_t)batch * 4, cudaMemcpyHostToDevice));
    for (int i = 0; i < batch; i++) D->pos_hi[(size_t)i] = positions_host[i];
    return TLC_OK;
}

extern "C" int32_t tlc_decoder_decode_enqueue(tlc_decoder *D, int32_t batch, int32_t steps) {
    TLC_REQUIRE(D, TLC_ERR_INVALID_OPERATION, "decoder_decode: null handle");
    if (int32_t rc = tlc_enter(D->ctx)) return rc;
    TLC_REQUIRE(batch >= 1 && batch <= D->cfg.max_batch, TLC_ERR_SHAPE_MISMATCH, "batch %d (max %d)", batch, D->cfg.max_batch);
    TLC_REQUIRE(steps >= 0, TLC_ERR_INVALID_OPERATION, "decode of %d steps", steps);
    if (int32_t rc = reserve_positions(D, batch, steps)) return rc;
    if (steps == 0) return TLC_OK;
    if (!D->cfg.no_graph)
        if (int32_t rc = step_graph(D, batch, batch)) return rc;
    for (int s = 0; s < steps; s++) {
        if (D->cfg.no_graph) {
            const uint64_t before = D->ctx->launches;
            if (int32_t rc = decode_step(D, batch, true)) return rc;
            D->launches = (int)(D->ctx->launches - before);
        } else {
            TLC_CUDA(cudaGraphLaunch(D->graph[batch], D->ctx->stream));
            D->ctx->launches += (uint64_t)D->launches;
        }
    }
    return TLC_OK;
}

extern "C" int32_t tlc_decoder_decode_host(tlc_decoder *D, int32_t batch, const int32_t *ids_host, int32_t *next_ids_host,
                                           float *logits_host) {
    TLC_REQUIRE(D && next_ids_host, TLC_ERR_INVALID_OPERATION, "decoder_decode_host: null pointer");
    tlc_ctx *ctx = D->ctx;
    if (int32_t rc = tlc_enter(ctx)) return rc;
    tlc_perf_scope perf(ctx, "decoder_decode(batch=%d)", batch);
    TLC_REQUIRE(batch >= 1 && batch <= D->cfg.max_batch, TLC_ERR_SHAPE_MISMATCH, "batch %d (max %d)", batch, D->cfg.max_batch);
    if (ids_host) {
        if (int32_t rc = check_ids(D, ids_host, batch)) return rc;
        memcpy(D->host_ids, ids_host, (size_t)batch * 4);
    }
    if (ids_host && !logits_host && !D->cfg.no_graph && ctx->host_graph) {
        // One graph launch: the gather reads the ids from pinned memory, the sampling kernel writes
        // the status word and the sampled ids there, the host watches those words.
        if (int32_t rc = reserve_positions(D, batch, 1)) return rc;
        D->ids_src = D->host_ids;
        D->report = HostReport{D->host_next, ctx->host_status, ctx->dev_status};
        const int32_t rc = step_graph(D, batch, 1000 + batch);
        D->ids_src = nullptr;
        D->report = HostReport{};
        if (rc) return rc;
        volatile int32_t *landed = D->host_next;
        for (int i = 0; i < batch; i++) landed[i] = -1;  // no token id is negative
        TLC_CUDA(cudaGraphLaunch(D->graph[1000 + batch], ctx->stream));
        ctx->launches += (uint64_t)D->launches;
        bool seen = false;
        if (ctx->host_poll) {
            const auto t0 = std::chrono::steady_clock::now();
            for (long spin = 0; !seen; spin++) {
                seen = true;
                for (int i = 0; i < batch; i++) seen = seen && landed[i] >= 0;
                if (!seen && (spin & 1023) == 1023 && std::chrono::steady_clock::now() - t0 > std::chrono::milliseconds(50)) break;
            }
        }
        if (!seen) TLC_CUDA(cudaStreamSynchronize(ctx->stream));
        if (int32_t rc2 = tlc_status_after_sync(ctx)) return rc2;
        memcpy(next_ids_host, D->host_next, (size_t)batch * 4);
        return TLC_OK;
    }
    if (ids_host) TLC_CUDA(cudaMemcpyAsync(D->ids, D->host_ids, (size_t)batch * 4, cudaMemcpyHostToDevice, ctx->stream));
    if (int32_t rc = tlc_decoder_decode_enqueue(D, batch, 1)) return rc;
    if (logits_host)
        TLC_CUDA(cudaMemcpyAsync(logits_host, D->logits, (size_t)batch * D->cfg.vocab * 4, cudaMemcpyDeviceToHost, ctx->stream));
    TLC_CUDA(cudaMemcpyAsync(D->host_next, D->next_ids, (size_t)batch * 4, cudaMemcpyDeviceToHost, ctx->stream));
    if (int32_t rc = tlc_synchronize(ctx)) return rc;
    memcpy(next_ids_host, D->host_next, (size_t)batch * 4);
    return TLC_OK;
}

extern "C" int32_t tlc_decoder_read_state(tlc_decoder *D, int32_t batch, int32_t *next_ids_host, int32_t *positions_host) {
    TLC_REQUIRE(D, TLC_ERR_INVALID_OPERATION, "decoder_read_state: null handle");
    TLC_REQUIRE(batch >= 1 && batch <= D->cfg.max_batch, TLC_ERR_SHAPE_MISMATCH, "batch %d (max %d)", batch, D->cfg.max_batch);
    if (next_ids_host)
        if (int32_t rc = tlc_download(D->ctx, next_ids_host, D->next_ids, (size_t)batch * 4)) return rc;
    if (positions_host)
        if (int32_t rc = tlc_download(D->ctx, positions_host, D->positions, (size_t)batch * 4)) return rc;
    return TLC_OK;
}

extern "C" int32_t tlc_decoder_set_sampling(tlc_decoder *D, float temperature, uint64_t seed) {
    TLC_REQUIRE(D, TLC_ERR_INVALID_OPERATION, "decoder_set_sampling: null handle");
    TLC_REQUIRE(temperature >= 0.f && temperature == temperature, TLC_ERR_INVALID_OPERATION, "temperature must be >= 0 (got %f)",
                (double)temperature);
    if (int32_t rc = tlc_enter(D->ctx)) return rc;
    TLC_CUDA(cudaStreamSynchronize(D->ctx->stream));
    drop_graphs(D);  // they hold the old sampling kernel and its arguments
    D->temperature = temperature;
    D->seed = seed;
    return TLC_OK;
}

extern "C" int32_t tlc_decoder_launches_per_step(tlc_decoder *D) { return D ? D->launches : 0; }
extern "C" tlc_kvcache *tlc_decoder_cache(tlc_decoder *D) { return D ? D->cache : nullptr; }
