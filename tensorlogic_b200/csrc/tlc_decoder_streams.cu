// Layers over several residual streams (hyper-connections) with latent attention, of the config-driven
// decoder.
//
// The norm between sublayers is element by element, so the projection that ends a sublayer also updates
// the streams and writes the next sublayer's normalized input (StreamsOut): no kernel touches the
// streams on its own except the embedding and, for the wanted rows of a portion, the last norm.
//   one row, seven launches per layer:
//     [W_dq, W_dkv] [query: norm, W_uq, rotation, q' = W_uk^T q; append] [scan of the cache]
//     [merge, sink, W_uv] [W_o -> streams, h] [gate, up] [down -> streams, h]
//   many rows:
//     [W_dq, W_dkv] [norms, rotation, append] then
//       long portions:  [W_uq; keys and values of the whole stretch from the cache] [attention]
//       batches, short: [W_uq] [q'] [scan] [merge, sink, W_uv]
//     [W_o -> streams, h] [gate, up] [down -> streams, h]
#include <algorithm>
#include <cmath>

#include "tlc_decoder.h"

extern "C" int32_t tlc_model_get(tlc_model *, const char *, tlc_qtensor **);
extern "C" int32_t tlc_kvcache_layer_ptrs(tlc_kvcache *, int32_t, void **, void **);

namespace tlc_dense {

namespace {

constexpr int kAbsorbRows = 16;  // portions of up to so many rows read the cache's latents as they are

// Values of a small tensor on the host.
int32_t host_values(tlc_decoder *D, const tlc_qtensor *t, std::vector<float> *out) {
    std::vector<uint8_t> raw((size_t)t->n_rows * t->row_pitch);
    TLC_CUDA(cudaMemcpyAsync(raw.data(), t->data, raw.size(), cudaMemcpyDeviceToHost, D->ctx->stream));
    TLC_CUDA(cudaStreamSynchronize(D->ctx->stream));
    out->clear();
    for (int64_t r = 0; r < t->n_rows; r++)
        for (int64_t c = 0; c < t->n_cols; c++) {
            const uint8_t *at = raw.data() + r * t->row_pitch + c * D->elem;
            if (D->elem == 4) {
                float v;
                memcpy(&v, at, 4);
                out->push_back(v);
            } else {
                uint16_t b;
                memcpy(&b, at, 2);
                const uint32_t u = (uint32_t)b << 16;
                float v;
                memcpy(&v, &u, 4);
                out->push_back(v);
            }
        }
    return TLC_OK;
}

bool expands(const tlc_decoder *D, const tlc_decoder_layer &c) {
    return D->cfg.dtype == TLC_TYPE_BF16 && latent_prefill_fits(c.dim, c.rot_dims, c.vdim, c.scale);
}

// The streams' update behind sublayer q of `L`, with the next sublayer's norm; h: its input or null.
StreamsOut streams_out(tlc_decoder *D, const StreamLayer &L, int q, const StreamSublayer *next, void *h) {
    StreamsOut o{};
    const int S = D->cfg.streams;
    o.x = D->st.x;
    o.plane = (int64_t)D->rows * D->cfg.width;
    o.n = S;
    const StreamSublayer &s = L.sub[q];
    for (int a = 0; a < S; a++) {
        o.out[a] = s.out[(size_t)a];
        o.in[a] = next ? next->in[(size_t)a] : 1.f;
        for (int b = 0; b < S; b++) o.mix[a][b] = s.mix[(size_t)a * S + b];
    }
    const StreamNorm &n = next ? next->norm : D->st.final_norm;
    o.alpha = n.alpha;
    o.scale = s.scale->data;
    o.w = n.w->data;
    o.b = n.b->data;
    o.h = h;
    o.ldh = D->ldw;
    return o;
}

// The sublayer that runs after sublayer q of run r, or null at the end.
const StreamSublayer *next_sublayer(const tlc_decoder *D, size_t r, int q) {
    const StreamLayer &L = D->st.layers[(size_t)D->runs[r]];
    if (q == 0 && L.c.ff_kind != TLC_FF_NONE) return &L.sub[1];
    return r + 1 < D->runs.size() ? &D->st.layers[(size_t)D->runs[r + 1]].sub[0] : nullptr;
}

template <typename T>
LatentParams latent_params(tlc_decoder *D, const StreamLayer &L, int run, const Pass &ps) {
    const tlc_decoder_layer &c = L.c;
    const int es = (int)sizeof(T);
    LatentParams p{};
    p.H = c.heads;
    p.D = c.dim;
    p.R = c.rot_dims;
    p.V = c.vdim;
    p.QR = c.q_rank;
    p.KR = c.kv_rank;
    p.kp = L.kp;
    p.row = L.row;
    p.m = ps.m;
    p.max_seq = D->cfg.max_seq;
    p.eps = D->cfg.norm_eps;
    p.scale = c.scale;
    p.dq_norm = L.dqn->data;
    p.dkv_norm = L.dkvn->data;
    p.sink = L.sink->data;
    p.uq = L.uq->data;
    p.uk = L.uk->data;
    p.uv = L.uv->data;
    p.uq_pitch = (int)(L.uq->row_pitch / es);
    p.uk_pitch = (int)(L.uk->row_pitch / es);
    p.uv_pitch = (int)(L.uv->row_pitch / es);
    p.freq = L.freq;
    p.cq_raw = D->st.cq_raw;
    p.ckv_raw = D->st.ckv;
    p.ldcq = round8(c.q_rank);
    p.ldckv = round8(c.kv_rank + c.rot_dims);
    p.cq = D->st.cq;
    p.ldq = round8(c.heads * (c.dim + c.rot_dims));
    void *cache = nullptr;
    tlc_kvcache_layer_ptrs(D->cache, run, &cache, nullptr);
    p.cache = cache;
    p.pos = ps.pos;
    p.slot = ps.slot;
    p.ql = D->st.ql;
    p.part = D->st.part;
    p.stat = D->st.stat;
    p.out = D->st.attn;
    p.ldo = round8(c.heads * c.vdim);
    p.status = D->ctx->dev_status;
    p.wait_ns = D->ctx->wait_ns;
    p.nsplit = latent_splits(D->ctx, p);
    return p;
}

template <typename T>
int32_t layer_one_row(tlc_decoder *D, size_t r, const Pass &ps) {
    tlc_ctx *ctx = D->ctx;
    StreamsState &S = D->st;
    StreamLayer &L = S.layers[(size_t)D->runs[r]];
    const int w = D->cfg.width, es = (int)sizeof(T);
    auto segment = [&](GemvParams &g, const tlc_qtensor *t, void *out) -> GemvSeg & {
        GemvSeg &s = g.seg[g.n_seg++];
        s.w = t->data;
        s.out = out;
        s.n = (int)t->n_rows;
        s.epi = EPI_STORE;
        return s;
    };
    auto from_h = [&] {
        GemvParams g{};
        g.k = w;
        g.pitch = (int)(L.dq->row_pitch / es);
        g.xn = S.h;
        return g;
    };
    auto into_streams = [&](const tlc_qtensor *t, const void *in, const tlc_qtensor *bias, int q) {
        const StreamSublayer *next = next_sublayer(D, r, q);
        OutParams o{};
        o.seg[o.n_seg++] = {t->data, in, (int)t->n_cols, (int)(t->row_pitch / es), 0, 1, nullptr};
        o.bias = bias ? bias->data : nullptr;
        o.n = w;
        o.st = streams_out(D, L, q, next, next ? S.h : D->hf);
        return launch_out_gemv<T>(ctx, o);
    };
    GemvParams g = from_h();
    segment(g, L.dq, S.cq_raw);
    segment(g, L.dkv, S.ckv);
    if (int32_t rc = launch_gemv<T>(ctx, g)) return rc;
    const LatentParams p = latent_params<T>(D, L, (int)r, ps);
    if (int32_t rc = launch_latent_query<T>(ctx, p)) return rc;
    if (int32_t rc = launch_latent_absorbed<T>(ctx, p)) return rc;
    if (int32_t rc = into_streams(L.o, S.attn, nullptr, 0)) return rc;
    if (L.c.ff_kind == TLC_FF_NONE) return TLC_OK;
    g = from_h();
    GemvSeg &s = segment(g, L.gate, S.act);
    s.w2 = L.up->data;
    s.bias = L.gate_b->data;
    s.bias2 = L.up_b->data;
    s.epi = EPI_SILU_MUL;
    if (int32_t rc = launch_gemv<T>(ctx, g)) return rc;
    return into_streams(L.down, S.act, L.down_b, 1);
}

template <typename T>
int32_t layer_many_rows(tlc_decoder *D, size_t r, const Pass &ps, bool last_norm) {
    tlc_ctx *ctx = D->ctx;
    StreamsState &S = D->st;
    StreamLayer &L = S.layers[(size_t)D->runs[r]];
    const tlc_decoder_layer &c = L.c;
    const int w = D->cfg.width, m = ps.m;
    LatentParams p = latent_params<T>(D, L, (int)r, ps);
    {
        Gemm<T> g(D, m);
        g.operand(g.add(c.q_rank, EPI_STORE, S.cq_raw, p.ldcq), 0, S.a_h, S.h, D->ldw, L.m_dq, L.dq);
        g.operand(g.add(c.kv_rank + c.rot_dims, EPI_STORE, S.ckv, p.ldckv), 0, S.a_h, S.h, D->ldw, L.m_dkv, L.dkv);
        if (int32_t rc = g.launch()) return rc;
    }
    if (int32_t rc = launch_latent_rows<T>(ctx, p)) return rc;
    const bool expand = !ps.decode && m > kAbsorbRows && expands(D, c);
    {
        Gemm<T> g(D, m);
        g.operand(g.add((int)L.uq->n_rows, EPI_STORE, S.q, p.ldq), 0, L.a_cq, S.cq, p.ldcq, L.m_uq, L.uq);
        if (expand) {
            const int keys = ps.pos0 + m, row0 = ps.seq * D->cfg.max_seq;
            p.ldk = round8(c.heads * c.dim);
            p.ldv = S.ld_v;
            GemmGroup &k = g.add(c.heads * c.dim, EPI_STORE, S.k_all, p.ldk);
            g.operand(k, 0, S.a_cache[r], nullptr, 0, L.m_uk, L.uk);
            k.rows = keys;
            k.a_row0 = row0;
            // values transposed: rows of W_uv against rows of the cache
            GemmGroup &v = g.add(keys, EPI_STORE, S.v_all, p.ldv);
            g.operand(v, 0, L.m_uv, nullptr, 0, S.a_cache[r], L.uv);
            v.rows = c.heads * c.vdim;
            v.b_row0 = row0;
        }
        if (int32_t rc = g.launch()) return rc;
    }
    p.q = S.q;
    if (expand) {
        p.pos0 = ps.pos0;
        p.slot0 = ps.seq;
        p.k_all = S.k_all;
        p.v_all = S.v_all;
        p.q_map = D->maps + L.a_q;
        p.k_map = D->maps + L.a_k;
        p.v_map = D->maps + L.a_v;
        p.rot_map = D->maps + S.a_rot[r];
        if (int32_t rc = launch_latent_prefill(ctx, p)) return rc;
    } else {
        if (int32_t rc = launch_latent_query<T>(ctx, p)) return rc;
        if (int32_t rc = launch_latent_absorbed<T>(ctx, p)) return rc;
    }
    auto into_streams = [&](int a_map, const void *a, int lda, int b_map, const tlc_qtensor *t, const tlc_qtensor *bias, int q) {
        const StreamSublayer *next = next_sublayer(D, r, q);
        Gemm<T> g(D, m);
        GemmGroup &gr = g.add(w, EPI_STREAMS, nullptr, w);
        g.operand(gr, 0, a_map, a, lda, b_map, t);
        gr.bias = bias ? bias->data : nullptr;
        g.p.st = streams_out(D, L, q, next, next ? S.h : last_norm ? D->hf : nullptr);
        return g.launch();
    };
    if (int32_t rc = into_streams(L.a_attn, S.attn, p.ldo, L.m_o, L.o, nullptr, 0)) return rc;
    if (c.ff_kind == TLC_FF_NONE) return TLC_OK;
    {
        Gemm<T> g(D, m);
        GemmGroup &gr = g.add(c.ff, EPI_SILU_MUL, S.act, round8(c.ff));
        g.operand(gr, 0, S.a_h, S.h, D->ldw, L.m_gate, L.gate);
        gr.b2_map = L.m_up;
        gr.b2 = L.up->data;
        gr.bias = L.gate_b->data;
        gr.bias2 = L.up_b->data;
        if (int32_t rc = g.launch()) return rc;
    }
    return into_streams(L.a_act, S.act, round8(c.ff), L.m_down, L.down, L.down_b, 1);
}

template <typename T>
int32_t forward_t(tlc_decoder *D, const Pass &ps) {
    tlc_ctx *ctx = D->ctx;
    StreamsState &S = D->st;
    const int w = D->cfg.width;
    const StreamSublayer &first = S.layers[(size_t)D->runs[0]].sub[0];
    const StreamsOut start = streams_out(D, S.layers[(size_t)D->runs[0]], 0, &first, S.h);
    if (int32_t rc = launch_embed_streams<T>(ctx, D->embed, ps.ids, ps.m, start)) return rc;
    const bool one_row = ps.m == 1 && D->one_row_ok, all_rows = !ps.want && !ps.n_want;
    const int n = all_rows ? ps.m : ps.n_want;
    // the last norm: with the last projection when every row is wanted, else for the wanted rows alone
    const bool last_norm = one_row || all_rows;
    for (size_t r = 0; r < D->runs.size(); r++)
        if (int32_t rc = one_row ? layer_one_row<T>(D, r, ps) : layer_many_rows<T>(D, r, ps, last_norm)) return rc;
    if (n == 0) return TLC_OK;
    if (!last_norm) {
        const StreamsOut end = streams_out(D, S.layers[(size_t)D->runs[0]], 0, nullptr, D->hf);
        if (int32_t rc = launch_streams_norm<T>(ctx, end, w, ps.want, n)) return rc;
    }
    const int epi = D->cfg.logit_softcap > 0.f ? EPI_SOFTCAP_F32 : EPI_STORE_F32;
    if (n == 1 && gemv_fits(w)) {
        GemvParams g{};
        g.k = w;
        g.pitch = (int)(D->embed->row_pitch / sizeof(T));
        g.xn = D->hf;
        g.n_seg = 1;
        g.seg[0].w = D->embed->data;
        g.seg[0].out = D->logits;
        g.seg[0].n = D->cfg.vocab;
        g.seg[0].epi = epi;
        g.seg[0].limit = D->cfg.logit_softcap;
        return launch_gemv<T>(ctx, g);
    }
    Gemm<T> lm(D, n);
    GemmGroup &g = lm.add(D->cfg.vocab, epi, D->logits, D->cfg.vocab);
    lm.operand(g, 0, D->a_hf, D->hf, D->ldw, D->m_embed, D->embed);
    g.limit = D->cfg.logit_softcap;
    return lm.launch();
}

}  // namespace

int32_t check_stream_layer(const tlc_decoder_layer &c, int i) {
    TLC_REQUIRE(c.mixer == TLC_MIX_LATENT, TLC_ERR_INVALID_OPERATION, "layer %d: mixer %d does not run over several streams", i, c.mixer);
    TLC_REQUIRE(c.heads > 0 && c.heads <= 65534 && c.dim > 0 && c.vdim > 0 && c.q_rank > 0 && c.kv_rank > 0, TLC_ERR_INVALID_DIMENSION,
                "layer %d: %d heads of %d and %d values, latents of %d and %d", i, c.heads, c.dim, c.vdim, c.q_rank, c.kv_rank);
    TLC_REQUIRE(c.rot_dims >= 0 && c.rot_dims % 2 == 0 && (c.rot_dims == 0 || c.rot_base > 0), TLC_ERR_INVALID_DIMENSION,
                "layer %d: rotation of %d values, base %g", i, c.rot_dims, c.rot_base);
    TLC_REQUIRE(c.dim <= 4096 && c.vdim <= 4096 && c.rot_dims <= 4096 && c.kv_rank <= 8192 && c.q_rank <= 32768, TLC_ERR_INVALID_DIMENSION,
                "layer %d: heads or latents are too large", i);
    TLC_REQUIRE(c.ff_kind == TLC_FF_NONE || c.ff_kind == TLC_FF_SILU_GLU, TLC_ERR_INVALID_OPERATION,
                "layer %d: feed-forward %d does not run over several streams", i, c.ff_kind);
    if (c.ff_kind != TLC_FF_NONE) TLC_REQUIRE(c.ff > 0, TLC_ERR_INVALID_DIMENSION, "layer %d: feed-forward of width %d", i, c.ff);
    return TLC_OK;
}

int32_t bind_streams(tlc_decoder *D, tlc_model *model) {
    const tlc_decoder_config &cfg = D->cfg;
    const int64_t w = cfg.width, S = cfg.streams;
    auto get = [&](const std::string &name, int64_t rows, int64_t cols, tlc_qtensor **t) { return bind_tensor(D, model, name, rows, cols, t); };
    auto small = [&](const std::string &name, int64_t rows, int64_t cols, std::vector<float> *out) -> int32_t {
        tlc_qtensor *t = nullptr;
        if (int32_t rc = get(name, rows, cols, &t)) return rc;
        return host_values(D, t, out);
    };
    auto norm = [&](const std::string &name, StreamNorm &n) -> int32_t {
        if (int32_t rc = get(name, 1, w, &n.w)) return rc;
        if (int32_t rc = get(name + ".b", 1, w, &n.b)) return rc;
        std::vector<float> alpha;
        if (int32_t rc = small(name + ".alpha", 1, 1, &alpha)) return rc;
        n.alpha = alpha[0];
        return TLC_OK;
    };
    if (int32_t rc = get("embed", cfg.vocab, w, &D->embed)) return rc;
    if (int32_t rc = norm("final.norm", D->st.final_norm)) return rc;
    for (int i = 0; i < cfg.n_layers; i++) {
        StreamLayer &L = D->st.layers[(size_t)i];
        const tlc_decoder_layer &c = L.c;
        const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.", f = p + "mlp.";
        const int64_t H = c.heads, ff = c.ff;
        struct Want { tlc_qtensor **t; std::string n; int64_t r, c; };
        std::vector<Want> want = {{&L.dq, m + "dq", c.q_rank, w},
                                  {&L.dqn, m + "dq.norm", 1, c.q_rank},
                                  {&L.uq, m + "uq", H * (c.dim + c.rot_dims), c.q_rank},
                                  {&L.dkv, m + "dkv", c.kv_rank + c.rot_dims, w},
                                  {&L.dkvn, m + "dkv.norm", 1, c.kv_rank},
                                  {&L.uk, m + "uk", H * c.dim, c.kv_rank},
                                  {&L.uv, m + "uv", H * c.vdim, c.kv_rank},
                                  {&L.sink, m + "sink", 1, H},
                                  {&L.o, m + "o", w, H * c.vdim}};
        if (c.ff_kind != TLC_FF_NONE) {
            want.push_back({&L.gate, f + "gate", ff, w});
            want.push_back({&L.gate_b, f + "gate.b", 1, ff});
            want.push_back({&L.up, f + "up", ff, w});
            want.push_back({&L.up_b, f + "up.b", 1, ff});
            want.push_back({&L.down, f + "down", w, ff});
            want.push_back({&L.down_b, f + "down.b", 1, w});
        }
        const int subs = c.ff_kind != TLC_FF_NONE ? 2 : 1;
        for (int q = 0; q < subs; q++) want.push_back({&L.sub[q].scale, p + "ls" + std::to_string(q + 1), 1, w});
        for (Want &e : want)
            if (int32_t rc = get(e.n, e.r, e.c, e.t)) return rc;
        for (int q = 0; q < subs; q++) {
            const std::string hc = p + "hc" + std::to_string(q + 1) + ".";
            StreamSublayer &s = L.sub[q];
            if (int32_t rc = norm(p + "norm" + std::to_string(q + 1), s.norm)) return rc;
            if (int32_t rc = small(hc + "in", 1, S, &s.in)) return rc;
            if (int32_t rc = small(hc + "out", 1, S, &s.out)) return rc;
            if (int32_t rc = small(hc + "mix", S, S, &s.mix)) return rc;
        }
    }
    return TLC_OK;
}

int32_t prepare_streams(tlc_decoder *D, Maps &maps) {
    const tlc_decoder_config &cfg = D->cfg;
    StreamsState &S = D->st;
    const int w = cfg.width;
    const size_t R = (size_t)D->rows, es = D->elem, keys = (size_t)cfg.max_seq;
    size_t cq = 8, ckv = 8, q = 8, ql = 8, attn = 8, act = 8, k_all = 0, v_all = 0, part = 8, stat = 8;
    S.ld_v = round8(cfg.max_seq);
    for (StreamLayer &L : S.layers) {
        const tlc_decoder_layer &c = L.c;
        const bool expand = expands(D, c);
        // rows that may take the absorbed form
        const size_t A = expand ? std::min(R, (size_t)std::max(kAbsorbRows, cfg.max_batch)) : R;
        cq = std::max(cq, R * round8(c.q_rank));
        ckv = std::max(ckv, R * round8(c.kv_rank + c.rot_dims));
        q = std::max(q, R * round8(c.heads * (c.dim + c.rot_dims)));
        ql = std::max(ql, A * c.heads * L.row);
        attn = std::max(attn, R * round8(c.heads * c.vdim));
        act = std::max(act, R * round8(c.ff));
        if (expand) {
            k_all = std::max(k_all, keys * round8(c.heads * c.dim));
            v_all = std::max(v_all, (size_t)c.heads * c.vdim * S.ld_v);
        }
        LatentParams p{};
        p.H = c.heads;
        p.max_seq = cfg.max_seq;
        size_t stretches = 1;  // (row, stretch) pairs of a launch
        for (p.m = 1; p.m <= (int)A; p.m++) stretches = std::max(stretches, (size_t)p.m * latent_splits(D->ctx, p));
        part = std::max(part, stretches * c.heads * L.kp);
        stat = std::max(stat, stretches * c.heads * 2);
        // the one-row kernels keep their inputs in shared memory
        OutParams o{}, d{};
        o.n = d.n = w;
        o.seg[o.n_seg++].k = c.heads * c.vdim;
        d.seg[d.n_seg++].k = std::max(c.ff, 1);
        for (const OutParams &one : {o, d})
            if (!(D->elem == 4 ? layer_gemv_fits<float>(D->ctx, {}, one) : layer_gemv_fits<bf16>(D->ctx, {}, one))) D->one_row_ok = false;
        if (!gemv_fits(w)) D->one_row_ok = false;
        if (c.rot_dims > 0) {
            std::vector<float> fr((size_t)c.rot_dims / 2);
            for (size_t i = 0; i < fr.size(); i++) fr[i] = (float)std::pow(c.rot_base, -2.0 * (double)i / (double)c.rot_dims);
            if (int32_t rc = upload(D, &L.freq, fr.data(), fr.size() * 4)) return rc;
        }
    }
    struct { void **p; size_t bytes; } bufs[] = {
        {(void **)&S.x, (size_t)cfg.streams * R * w * 4},
        {(void **)&S.h, R * D->ldw * es},
        {(void **)&S.cq_raw, cq * es},
        {(void **)&S.cq, cq * es},
        {(void **)&S.ckv, ckv * es},
        {(void **)&S.q, q * es},
        {(void **)&S.ql, ql * es},
        {(void **)&S.attn, attn * es},
        {(void **)&S.act, act * es},
        {(void **)&S.k_all, k_all * es},
        {(void **)&S.v_all, v_all * es},
        {(void **)&S.part, part * 4},
        {(void **)&S.stat, stat * 4},
    };
    for (auto &b : bufs)
        if (int32_t rc = dev_alloc(D, b.p, b.bytes)) return rc;
    if (cfg.dtype != TLC_TYPE_BF16) return TLC_OK;
    S.a_h = maps.add(S.h, (int64_t)R, w, D->ldw);
    for (StreamLayer &L : S.layers) {
        const tlc_decoder_layer &c = L.c;
        L.m_dq = maps.weight(L.dq);
        L.m_uq = maps.weight(L.uq);
        L.m_dkv = maps.weight(L.dkv);
        L.m_uk = maps.weight(L.uk);
        L.m_uv = maps.weight(L.uv);
        L.m_o = maps.weight(L.o);
        L.a_cq = maps.add(S.cq, (int64_t)R, c.q_rank, round8(c.q_rank));
        L.a_attn = maps.add(S.attn, (int64_t)R, c.heads * c.vdim, round8(c.heads * c.vdim));
        if (L.gate) {
            L.m_gate = maps.weight(L.gate);
            L.m_up = maps.weight(L.up);
            L.m_down = maps.weight(L.down);
            L.a_act = maps.add(S.act, (int64_t)R, c.ff, round8(c.ff));
        }
        if (expands(D, c)) {
            const int qw = c.heads * (c.dim + c.rot_dims), kw = c.heads * c.dim;
            L.a_q = maps.add(S.q, (int64_t)R, qw, round8(qw));
            L.a_k = maps.add(S.k_all, cfg.max_seq, kw, round8(kw), 64);
            L.a_v = maps.add(S.v_all, (int64_t)c.heads * c.vdim, cfg.max_seq, S.ld_v, 64);
        }
    }
    for (size_t r = 0; r < D->runs.size(); r++) {
        const StreamLayer &L = S.layers[(size_t)D->runs[r]];
        void *cache = nullptr;
        tlc_kvcache_layer_ptrs(D->cache, (int32_t)r, &cache, nullptr);
        const int64_t rows = (int64_t)cfg.max_batch * cfg.max_seq;
        S.a_cache.push_back(maps.add(cache, rows, L.c.kv_rank, L.row));
        S.a_rot.push_back(L.c.rot_dims ? maps.add(static_cast<bf16 *>(cache) + L.kp, rows, L.c.rot_dims, L.row, 64) : -1);
    }
    return maps.bad;
}

int32_t forward_streams(tlc_decoder *D, const Pass &ps) {
    return D->cfg.dtype == TLC_TYPE_F32 ? forward_t<float>(D, ps) : forward_t<bf16>(D, ps);
}

}  // namespace tlc_dense
