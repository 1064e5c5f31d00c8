// Kernels over dense bf16 / f32 weights for the config-driven decoder: launch parameters and the
// device helpers the translation units share.  T is the type of weights, activations and cache;
// every sum, norm, angle, score, router value and the residual stream are f32.
//
// Launch order and programmatic dependent launch.  Every kernel of this family lets its successor
// be scheduled only after its own dependency wait (tlc_dense::pdl_enter).  A kernel can therefore
// not start before the predecessor of its predecessor is complete, and may read what older kernels
// wrote (positions, cache rows of earlier steps) before its own wait.  The one exception says so at
// its launch (expert_gemv_kernel).
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>

#include "tlc_internal.h"

namespace tlc_dense {

typedef __nv_bfloat16 bf16;

template <typename T>
struct Vec;  // values in 16 bytes
template <>
struct Vec<bf16> {
    static constexpr int N = 8;
};
template <>
struct Vec<float> {
    static constexpr int N = 4;
};

#ifdef __CUDACC__
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f32(float v) { return v; }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }

// The values of one 16-byte piece.
__device__ __forceinline__ void unpack(const uint4 &v, float (&f)[8]) {  // bf16
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        f[2 * i] = __uint_as_float(w[i] << 16);
        f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void unpack(const uint4 &v, float (&f)[4]) {  // f32
    f[0] = __uint_as_float(v.x);
    f[1] = __uint_as_float(v.y);
    f[2] = __uint_as_float(v.z);
    f[3] = __uint_as_float(v.w);
}

__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_enter() {
    pdl_wait();
    pdl_trigger();
}

__device__ __forceinline__ void prefetch_l2(const void *p, uint32_t bytes) {
    asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(p), "r"(bytes) : "memory");
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
// g = min(gate, limit), u = clamp(up, -limit, limit): g sigmoid(1.702 g) (u + 1)
__device__ __forceinline__ float clamped_glu(float gate, float up, float limit) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return g * sigmoid_f(1.702f * g) * (u + 1.0f);
}
__device__ __forceinline__ float silu_mul(float gate, float up) { return gate * sigmoid_f(gate) * up; }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Sum over the block, the same value in every thread; `red` holds 33 floats and may be used again
// after the next __syncthreads.
__device__ __forceinline__ float block_sum(float v, float *red) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    const int nw = (blockDim.x + 31) >> 5;
    float s = 0.f;
    for (int i = 0; i < nw; i++) s += red[i];
    return s;
}
#endif

// ---- what an epilogue does with a sum -----------------------------------------------------------
enum Epilogue {
    EPI_STORE = 0,        // out[row][n] = T(acc [+ bias])
    EPI_STORE_F32 = 1,    // out[row][n] = acc (f32)
    EPI_ADD_F32 = 2,      // out[row][n] += acc + bias (f32: the residual stream)
    EPI_SOFTCAP_F32 = 3,  // out[row][n] = limit * tanh(acc / limit) (f32)
    EPI_STREAMS = 4,      // y = (acc + bias) * scale into every residual stream (StreamsOut)
    EPI_CLAMPED_GLU = 5,  // pair: out = T(clamped_glu(gate, up) [* out_scale])
    EPI_SILU_MUL = 6,     // pair: out = T(silu(in_scale gate [+ bias]) (in_scale up [+ bias2]) [* out_scale])
};

// ---- several residual streams (hyper-connections) -----------------------------------------------
// The residual is n streams x_0 .. x_{n-1} (f32 planes).  A sublayer reads u = sum_s in[s] x_s through
// its norm and leaves x_t <- sum_s mix[s][t] x_s + out[t] y.  With a norm that needs no statistics of
// the row, tanh(alpha u) * w + b, everything behind the sublayer's last product is a function of one
// column: the projection that makes y updates the streams and stores the NEXT sublayer's input h.
constexpr int kMaxStreams = 8;
struct StreamsOut {
    float *x;               // [n][rows][width]: plane s starts at x + s * plane
    int64_t plane;
    int n;
    float out[kMaxStreams], mix[kMaxStreams][kMaxStreams];  // of this sublayer; mix[from][to]
    float in[kMaxStreams];  // of the next sublayer (all ones: the sum at the end)
    float alpha;            // next norm
    const void *scale;      // T [width]: multiplies y
    const void *w, *b;      // T [width]: next norm
    void *h;                // T [rows][ldh], or null: no next input is wanted
    int ldh;
};
#ifdef __CUDACC__
__device__ __forceinline__ float tanh_norm(float u, float alpha, float w, float b) { return tanhf(alpha * u) * w + b; }
// One column: `x` holds the old streams and receives the new ones; returns the next sublayer's u.  MAXS up to 4
// is the number of streams, larger only a bound.
template <int MAXS>
__device__ __forceinline__ int stream_count(const StreamsOut &o) {
    return MAXS <= 4 ? MAXS : o.n;
}
template <int MAXS>
__device__ __forceinline__ float update_streams(const StreamsOut &o, float y, float (&x)[MAXS]) {
    const int n = stream_count<MAXS>(o);
    float nw[MAXS], u = 0.f;
#pragma unroll
    for (int t = 0; t < MAXS; t++) {
        if (t >= n) continue;
        float v = o.out[t] * y;
#pragma unroll
        for (int s = 0; s < MAXS; s++)
            if (s < n) v = fmaf(o.mix[s][t], x[s], v);
        nw[t] = v;
        u = fmaf(o.in[t], v, u);
    }
#pragma unroll
    for (int t = 0; t < MAXS; t++)
        if (t < n) x[t] = nw[t];
    return u;
}
// The same with loads and stores, for column n of row `row` and the finished product `acc`.
template <typename T>
__device__ __forceinline__ void streams_column(const StreamsOut &o, int64_t row, int width, int n, float acc) {
    float x[kMaxStreams];
    float *at = o.x + row * width + n;
#pragma unroll
    for (int s = 0; s < kMaxStreams; s++)
        if (s < o.n) x[s] = __ldcg(at + s * o.plane);
    const float u = update_streams(o, acc * to_f32(static_cast<const T *>(o.scale)[n]), x);
#pragma unroll
    for (int s = 0; s < kMaxStreams; s++)
        if (s < o.n) at[s * o.plane] = x[s];
    if (o.h)
        static_cast<T *>(o.h)[row * o.ldh + n] =
            from_f32<T>(tanh_norm(u, o.alpha, to_f32(static_cast<const T *>(o.w)[n]), to_f32(static_cast<const T *>(o.b)[n])));
}
#endif

// ---- one activation row (decode): streams weight rows -------------------------------------------
// A segment of the output: n rows of a weight (pair: 2 n rows, gate and up alternating), all
// against the same input of K values.
struct GemvSeg {
    const void *w, *w2;  // w2: the up weight of a pair
    const void *bias;    // T [n] or null
    const void *bias2;   // T [n] or null: of the up weight
    void *out;
    int n;               // outputs
    int v0;              // first virtual row (even)
    int epi;             // Epilogue; pairs: EPI_CLAMPED_GLU or EPI_SILU_MUL
    int input;           // which normalized input: 0 or 1
    float limit;
};
struct GemvParams {
    GemvSeg seg[6];
    int n_seg, v_total;   // virtual rows, even per segment
    int k, pitch;         // inputs; elements between weight rows
    int split;            // stretches a row is cut into
    int rows_cap;         // virtual rows of the busiest CTA (size of the partial-sum area)
    const float *x;       // f32 [k]: layer-normalized here with norm_w[input]
    const void *xn;       // T [k], used as it is when not null
    const void *norm_w[2];
    float eps;
    float *h_out;         // f32 [k] or null: CTA 0 stores input 1 (the experts' input)
    int prefetch;         // weight rows of a CTA asked into the L2 before the dependency wait
};
template <typename T>
int32_t launch_gemv(tlc_ctx *ctx, GemvParams &p);

// Gate and up rows of the chosen experts of one token.
struct ExpertParams {
    const float *h;          // f32 [k]
    const float *logits;     // f32 [experts]
    const void *const *gate; // [experts] device pointers
    const void *const *up;
    void *act;               // T [top][act_pitch]
    int *chosen;             // [top], written by CTA 0
    float *weight;           // [top]
    int experts, top, k, pitch, ff, act_pitch, split, rows_cap;
};
template <typename T>
int32_t launch_expert_gemv(tlc_ctx *ctx, ExpertParams &p);

// x[n] += bias[n] + sum over segments of scale * (w[n] . input)
struct OutSeg {
    const void *w;
    const void *in;       // T [k]
    int k, pitch, c0;     // c0: first 16-byte piece in the concatenation
    int split;            // stretches a row is cut into
    const float *scale_logit;  // or null: the segment counts times sigmoid(*scale_logit)
};
struct OutParams {
    OutSeg seg[2];
    int n_seg;
    const void *const *down;  // experts' weights or null
    const int *chosen;
    const void *expert_in;    // T [top][expert_in_pitch]
    int top, expert_k, expert_pitch, expert_in_pitch, expert_c0, expert_pieces;
    const void *bias;         // T [n] or null
    float *x;
    int n, pieces;            // 16-byte pieces of the whole concatenation
    int expert_split, rows_cap, prefetch;
    StreamsOut st;            // st.n > 0: the sums go into the streams instead of x (without experts)
};
template <typename T>
int32_t launch_out_gemv(tlc_ctx *ctx, OutParams &p);

// Do the inputs of these launches fit the shared memory?  (Sizes only: pointers may be null.)
bool gemv_fits(int k);
template <typename T>
bool layer_gemv_fits(const tlc_ctx *ctx, ExpertParams e, OutParams o);

// ---- many activation rows ------------------------------------------------------------------------
struct GemmGroup {
    // one or two stretches of K that add up (the second: k[1] > 0)
    int a_map[2], b_map[2], b2_map;      // tensor maps (bf16 form); b2_map: the up weight of a pair, else -1
    const void *a[2], *b[2], *b2;        // the same operands as pointers (f32 form)
    int lda[2], ldb[2], k[2];
    int n, epi;
    int rows, a_row0, b_row0;  // dense groups: rows of A (and out), where they start in A's map and where B's do
    const void *bias, *bias2;  // bias2: of the up weight
    void *out;
    int ldo;
    float limit;
    const float *in_scale;   // f32 per row of A, or null
    const float *out_scale;  // f32 [row * out_scale_stride], sigmoid applied, or null
    int out_scale_stride;
    // experts > 0: rows off[e] .. off[e + 1] of A and out belong to weight e, whose maps are
    // b_map[0] + e * map_stride and b2_map + e * map_stride and whose pointers are b_tab[e], b2_tab[e]
    int experts, map_stride;
    int in_rows_per_token;   // a family: rows of A per token (choices of the router)
    const int *off;
    const void *const *b_tab, *const *b2_tab;
};
struct GemmParams {
    GemmGroup g[6];
    int n_groups, m;
    int slots;  // dense groups + experts of all families
    const CUtensorMap *maps;
    tlc_dev_status *status;
    uint64_t wait_ns;
    StreamsOut st;  // of the EPI_STREAMS group (at most one)
};
constexpr int kMaxSlots = 1100;
// bf16: tcgen05; f32: FMA pipes, no reduced precision.
template <typename T>
int32_t launch_gemm(tlc_ctx *ctx, GemmParams &p);
// Tensor map of a row-major bf16 matrix in boxes of `box_rows` (at most 256) rows x 64 columns.
int32_t encode_map(CUtensorMap *map, const void *base, int64_t rows, int64_t cols, int64_t pitch, int box_rows = 128);

// ---- norms, rotation, routing --------------------------------------------------------------------
template <typename T>
int32_t launch_embed(tlc_ctx *ctx, const tlc_qtensor *table, const int *ids, int m, float *x);

// Several streams: every plane of `st` gets the embedding rows; h receives norm(sum(in) * row).
template <typename T>
int32_t launch_embed_streams(tlc_ctx *ctx, const tlc_qtensor *table, const int *ids, int m, const StreamsOut &st);
// h[i] = norm(sum_s in[s] x_s[rows[i]]) for m rows (rows null: i itself).
template <typename T>
int32_t launch_streams_norm(tlc_ctx *ctx, const StreamsOut &st, int width, const int *rows, int m);

// Layer norms of the rows of x; a pending sum of expert outputs is added to x first.
struct NormParams {
    float *x;
    int m, d;
    const int *rows;        // null: row i of x is row i; else x row rows[i] gives output row i
    const void *y;          // T [pairs][y_pitch] expert outputs or null
    const int *place;       // [x row][top]: rows of y
    int top, y_pitch;
    const void *w[2];       // w[1] may be null
    void *out[2];           // T
    int ldo;
    float eps;
    int *zero;              // ints cleared for the router, or null
    int n_zero;
};
template <typename T>
int32_t launch_norm(tlc_ctx *ctx, const NormParams &p);

struct RotParams {
    const void *q, *k;        // raw projections T [m][ldq], [m][ldk]
    int ldq, ldk;
    const void *qn, *kn;      // norm weights T
    const float *freq;        // [rot / 2]
    int H, G, D, Dp, rot;     // Dp: padded row of a head
    float eps;
    const int *pos, *slot;
    int max_seq;
    void *q_out;              // T [m][H][Dp]
    void *kc, *vc;            // this layer's cache [slot][max_seq][G][Dp]
    tlc_dev_status *status;
};
template <typename T>
int32_t launch_qk_rotate(tlc_ctx *ctx, const RotParams &p, int m);

struct RouteParams {
    const float *logits;    // [m][ld]
    int ld, experts, top, m;
    int *chosen, *rank, *count;  // [m][top], [m][top], [experts] (zero on entry)
    float *weight;               // [m][top]
};
int32_t launch_route(tlc_ctx *ctx, const RouteParams &p);
struct PermuteParams {
    const void *h;          // T [m][ldh]
    int m, d, ldh, top, experts;
    const int *chosen, *rank, *count;
    const float *weight;
    int *off;               // [experts + 1]
    int *place;             // [m][top]
    void *hp;               // T [m * top][ldh]
    float *scale;           // [m * top]
};
template <typename T>
int32_t launch_permute(tlc_ctx *ctx, const PermuteParams &p);

// ---- windowed attention ---------------------------------------------------------------------------
struct WindowAttn {
    const void *q;            // prepared: T [m][H][Dp]; raw (fused decode): T [m][ldq]
    const void *k_raw;        // fused decode: T [m][ldk]
    int ldq, ldk;
    const void *qn, *kn;
    const float *freq;
    int rot;
    float eps;
    void *kc, *vc;
    void *out;                // T [m][ldo], head h at h * D
    int ldo;
    int H, G, D, Dp;
    int window, keep;
    float scale;
    const int *pos, *slot;
    int max_seq;
    int m;
    int pos0;                 // prefill: position of row 0 (rows are consecutive, one slot)
    int nsplit;               // decode: CTAs per (row, kv head, 16 heads)
    tlc_dev_status *status;
};
// Rows of one sequence at consecutive positions, keys and queries prepared (bf16).
int32_t launch_window_prefill(tlc_ctx *ctx, const WindowAttn &p, int slot);
// One query per row, every row another sequence: norms, rotation, cache append and attention in one launch (bf16).
int32_t launch_window_decode(tlc_ctx *ctx, WindowAttn p);
// Any rows, any size of head up to 512, keys and queries prepared.
template <typename T>
int32_t launch_window_rows(tlc_ctx *ctx, const WindowAttn &p);
bool window_tensor_cores(int D);

// ---- latent attention ------------------------------------------------------------------------------
// Keys and values of all heads are projections of one latent c (size KR) per token, plus one rotated key
// part (size R) all heads share; the cache holds rows [c, 0.. | rotated part, 0..] of `row` values, the
// rotated part at kp.  Two forms of the same scores:
//   absorbed  q' = W_uk^T q per head, scores q'.c + q_rot.k_rot, values c, W_uv applied to the weighted
//             latent: the cache is read once for all heads (decode, short portions, every f32 pass);
//   expanded  keys W_uk c and values W_uv c are made for a stretch of the cache first (long portions).
// Softmax: one more term exp(sink[head]) in the denominator.
struct LatentParams {
    int H, D, R, V, QR, KR;   // heads; unrotated, rotated, value size per head; query and key/value latent
    int kp, row;              // KR padded to 8; values of a cache row
    int m, max_seq;
    float eps, scale;
    const void *dq_norm, *dkv_norm, *sink;  // T
    const void *uq, *uk, *uv;               // T, rows of *_pitch values
    int uq_pitch, uk_pitch, uv_pitch;
    const float *freq;        // [R / 2]
    const void *cq_raw;       // T [m][ldcq]: W_dq h
    const void *ckv_raw;      // T [m][ldckv]: W_dkv h
    int ldcq, ldckv;
    void *cq;                 // T [m][ldcq]: normalized (many rows)
    const void *q;            // T [m][ldq]: W_uq cq (many rows; null: the query kernel makes it)
    int ldq;
    void *cache;              // T [slot][max_seq][row]
    const int *pos, *slot;
    void *ql;                 // T [m][H][row]: absorbed queries
    float *part, *stat;       // [m][nsplit][H][kp]; [m][H][nsplit][2]: maximum (base 2) and sum
    int nsplit;
    void *out;                // T [m][ldo], head h at h * V
    int ldo;
    // expanded
    const void *k_all;        // bf16 [keys][ldk]: unrotated keys, head h at h * D
    const void *v_all;        // bf16 [H * V][ldv]: values, transposed
    int ldk, ldv;
    int pos0, slot0;          // rows are consecutive positions from pos0 of sequence slot0
    const CUtensorMap *q_map, *k_map, *v_map, *rot_map;  // of q, k_all, v_all, the cache's rotated parts
    tlc_dev_status *status;
    uint64_t wait_ns;
};
// Many rows: latents normalized and appended to the cache, query latents normalized into cq.
template <typename T>
int32_t launch_latent_rows(tlc_ctx *ctx, const LatentParams &p);
// Absorbed queries.  p.q null (one row): also the norms, W_uq and the cache append.
template <typename T>
int32_t launch_latent_query(tlc_ctx *ctx, const LatentParams &p);
// Attention over the cache in p.nsplit stretches, then merge, sink and W_uv.
template <typename T>
int32_t launch_latent_absorbed(tlc_ctx *ctx, const LatentParams &p);
int latent_splits(const tlc_ctx *ctx, const LatentParams &p);  // stretches for p.m rows of p.H heads
// Expanded: attention of consecutive rows over k_all, v_all and the cache's rotated parts (bf16).
int32_t launch_latent_prefill(tlc_ctx *ctx, const LatentParams &p);
bool latent_prefill_fits(int D, int R, int V, float scale);

}  // namespace tlc_dense
