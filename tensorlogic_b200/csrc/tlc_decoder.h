// The config-driven decoder's state, shared by its translation units: tlc_decoder.cu (the runner, and
// layers whose branches read one residual) and tlc_decoder_streams.cu (layers over several residual
// streams).
#pragma once

#include <cstring>

#include "tlc_dense.cuh"
#include "tlc_sample.cuh"

namespace tlc_dense {

constexpr int kMaxSeqs = 64;
inline int round8(int n) { return (n + 7) & ~7; }

struct Layer {
    tlc_decoder_layer c;
    tlc_qtensor *norm1 = nullptr, *norm2 = nullptr;
    tlc_qtensor *q, *qb, *qn, *k, *kb, *kn, *o, *ob;
    tlc_qtensor *gate = nullptr, *up = nullptr, *down = nullptr;  // dense or shared expert
    tlc_qtensor *router = nullptr, *sg = nullptr;
    std::vector<tlc_qtensor *> e_gate, e_up, e_down;
    float *freq = nullptr;                                           // [rot_dims / 2]
    const void **gate_tab = nullptr, **up_tab = nullptr, **down_tab = nullptr;  // device, per expert
    // tensor maps by index (bf16)
    int m_q = -1, m_k = -1, m_o = -1, m_gate = -1, m_up = -1, m_down = -1, m_router = -1, m_sg = -1;
    int m_egate = -1, m_eup = -1, m_edown = -1;
    int a_attn = -1, a_act = -1, a_acte = -1;                        // activations of this layer's widths
    int ff_width() const { return c.ff_kind == TLC_FF_MOE ? c.shared_ff : c.ff_kind ? c.ff : 0; }
};

// A layer over several streams: latent attention, then a feed-forward or none.
struct StreamNorm {
    tlc_qtensor *w = nullptr, *b = nullptr;
    float alpha = 0.f;
};
struct StreamSublayer {  // how a sublayer reads and writes the streams
    StreamNorm norm;
    tlc_qtensor *scale = nullptr;
    std::vector<float> in, out, mix;
};
struct StreamLayer {
    tlc_decoder_layer c;
    StreamSublayer sub[2];  // mixer, feed-forward
    tlc_qtensor *dq, *dqn, *uq, *dkv, *dkvn, *uk, *uv, *sink, *o;
    tlc_qtensor *gate = nullptr, *gate_b = nullptr, *up = nullptr, *up_b = nullptr, *down = nullptr, *down_b = nullptr;
    float *freq = nullptr;  // [rot_dims / 2]
    int kp = 0, row = 0;    // cache row: the latent in kp values, then the rotated part
    // tensor maps by index (bf16)
    int m_dq = -1, m_uq = -1, m_dkv = -1, m_uk = -1, m_uv = -1, m_o = -1, m_gate = -1, m_up = -1, m_down = -1;
    int a_cq = -1, a_attn = -1, a_act = -1, a_q = -1, a_k = -1, a_v = -1;
};
struct StreamsState {
    std::vector<StreamLayer> layers;
    StreamNorm final_norm;
    float *x = nullptr;     // [streams][rows][width]
    uint8_t *h = nullptr, *cq_raw = nullptr, *cq = nullptr, *ckv = nullptr, *q = nullptr, *ql = nullptr, *attn = nullptr, *act = nullptr;
    uint8_t *k_all = nullptr, *v_all = nullptr;  // expanded keys and transposed values of one layer
    int ld_v = 0;
    float *part = nullptr, *stat = nullptr;
    int a_h = -1, a_hf = -1;
    std::vector<int> a_cache, a_rot;  // per run: the cache's latents, its rotated parts
};

}  // namespace tlc_dense

struct tlc_decoder {
    tlc_ctx *ctx;
    tlc_decoder_config cfg;
    std::vector<tlc_dense::Layer> layers;
    tlc_dense::StreamsState st;   // cfg.streams > 0
    std::vector<int> runs;        // layer numbers in the order they run
    tlc_qtensor *embed, *final_norm;
    tlc_kvcache *cache = nullptr;
    size_t elem;
    int rows, logit_rows, top_max = 0;
    bool one_row_ok = true;     // every layer's inputs fit the one-row kernels
    std::vector<void *> owned;  // device allocations
    CUtensorMap *maps = nullptr;
    int a_h1 = -1, a_h2 = -1, a_hp = -1, a_hf = -1, m_embed = -1;
    // activations
    float *x, *h_row, *router_out, *weight, *scale, *logits;
    uint8_t *h1, *h2, *q_raw, *k_raw, *q_rot, *attn, *act, *hp, *act_e, *y, *hf;
    int ldw, ld_router = 1;
    int *chosen, *rank, *place, *count, *off;
    // row metadata: of a prompt portion, and of the sequences (decode)
    int *row_ids, *row_pos, *row_slot, *want;
    int *ids, *positions, *next_ids, *slots;
    int *host_rows = nullptr;     // pinned: ids, positions, slots, wanted rows
    int *host_next = nullptr;     // pinned
    int *host_ids = nullptr;      // pinned
    const int *ids_src = nullptr; // set while the host step is captured
    HostReport report{};
    std::map<int, cudaGraphExec_t> graph;  // batch; 1000 + batch: the host step
    int launches = 0;
    std::vector<int> pos_hi;      // host-side upper bound of every sequence's position
    float temperature = 0.f;
    uint64_t seed = 0;
};

namespace tlc_dense {

// Device memory the decoder owns, zero-filled: padding columns are read as zeros.
int32_t dev_alloc(tlc_decoder *D, void **p, size_t bytes);
// The model's tensor `name`, of this shape and of the type the decoder runs in.
int32_t bind_tensor(tlc_decoder *D, tlc_model *model, const std::string &name, int64_t rows, int64_t cols, tlc_qtensor **t);

template <typename P>
int32_t upload(tlc_decoder *D, P **dst, const void *src, size_t bytes) {
    void *p = nullptr;
    if (int32_t rc = dev_alloc(D, &p, bytes)) return rc;
    TLC_CUDA(cudaMemcpyAsync(p, src, bytes, cudaMemcpyHostToDevice, D->ctx->stream));
    TLC_CUDA(cudaStreamSynchronize(D->ctx->stream));  // `src` may go away
    *dst = static_cast<P *>(p);
    return TLC_OK;
}

// What one pass computes.
struct Pass {
    int m;                  // rows
    const int *ids, *pos, *slot;
    bool decode;            // every row is another sequence
    int seq = 0, pos0 = 0;  // portion: its sequence and the position of row 0
    const int *want = nullptr;  // device: rows whose logits are computed, or null: all m rows
    int n_want = 0;
    int want_single = -1;   // the row, when n_want == 1 and it is known on the host
};

template <typename T>
struct Gemm {  // builds one grouped launch
    tlc_decoder *D;
    GemmParams p{};
    Gemm(tlc_decoder *d, int m) : D(d) {
        p.m = m;
        p.maps = d->maps;
    }
    GemmGroup &add(int n, int epi, void *out, int ldo) {
        GemmGroup &g = p.g[p.n_groups++];
        g = GemmGroup{};
        g.n = n;
        g.rows = p.m;
        g.epi = epi;
        g.out = out;
        g.ldo = ldo;
        g.b2_map = -1;
        return g;
    }
    void operand(GemmGroup &g, int seg, int a_map, const void *a, int lda, int b_map, const tlc_qtensor *b) {
        g.a_map[seg] = a_map;
        g.a[seg] = a;
        g.lda[seg] = lda;
        g.b_map[seg] = b_map;
        g.b[seg] = b->data;
        g.ldb[seg] = (int)(b->row_pitch / sizeof(T));
        g.k[seg] = (int)b->n_cols;
    }
    int32_t launch() { return launch_gemm<T>(D->ctx, p); }
};

// Tensor maps collected on the host (bf16).
struct Maps {
    std::vector<CUtensorMap> maps;
    int32_t bad = TLC_OK;
    int add(const void *base, int64_t rows, int64_t cols, int64_t pitch, int box_rows = 128) {
        CUtensorMap m;
        if (!bad) bad = encode_map(&m, base, rows, cols, pitch, box_rows);
        maps.push_back(m);
        return (int)maps.size() - 1;
    }
    int weight(const tlc_qtensor *t) { return add(t->data, t->n_rows, t->n_cols, (int64_t)(t->row_pitch / 2)); }
};

// Layers over several streams (tlc_decoder_streams.cu).
int32_t check_stream_layer(const tlc_decoder_layer &c, int i);
int32_t bind_streams(tlc_decoder *D, tlc_model *model);
int32_t prepare_streams(tlc_decoder *D, Maps &maps);
int32_t forward_streams(tlc_decoder *D, const Pass &ps);

}  // namespace tlc_dense
