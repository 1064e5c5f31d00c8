// One activation row against dense weights: the decode step of one sequence.
//
// Three kernels, one launch each:
//   gemv_kernel         layer norm(s) of the residual row, then several weights against the
//                       normalized inputs (q, k, gate/up pairs, router, lm_head);
//   expert_gemv_kernel  router decision, then gate/up of the chosen experts;
//   out_gemv_kernel     the projections back into the residual stream -- attention output,
//                       feed-forward down, chosen experts, shared expert -- as ONE sum per output.
// All are bound by the weights' bytes.  A warp streams stretches of weight rows in 16-byte loads that
// roll on from one stretch to the next, so that a lane always has the same number in flight; CTAs own
// contiguous rows, the partial sums meet in shared memory after the last load, so no barrier
// interrupts the stream.  The input sits in shared memory as f32, unrounded.
#include <cstring>

#include "tlc_dense.cuh"
#include "tlc_stream.cuh"

namespace tlc_dense {

namespace {

constexpr int kThreads = 512, kWarps = kThreads / 32;
constexpr size_t kSmemMax = 200 * 1024;

template <typename T>
__global__ void __launch_bounds__(kThreads, 2) gemv_kernel(const __grid_constant__ GemvParams p) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float red[33];
    const int tid = threadIdx.x;
    const int pieces = (p.k + Vec<T>::N - 1) / Vec<T>::N;
    const int row_floats = pieces * Vec<T>::N;
    float *xs[2] = {smem, smem + row_floats};
    uint4 *nw = reinterpret_cast<uint4 *>(smem + 2 * (size_t)row_floats);  // the two norm weights, [2][pieces]
    float *part = reinterpret_cast<float *>(nw + (p.xn ? 0 : 2 * pieces));

    // virtual rows of this CTA, cut at even numbers
    const int pairs = p.v_total >> 1;
    const int v_lo = 2 * (int)((long long)pairs * blockIdx.x / gridDim.x);
    const int v_hi = 2 * (int)((long long)pairs * (blockIdx.x + 1) / gridDim.x);
    auto find = [&](int v) {
        int s = 0;
        while (s + 1 < p.n_seg && v >= p.seg[s + 1].v0) s++;
        return s;
    };
    auto weight_row = [&](int s, int v) -> const T * {  // null: the padding row of an odd segment
        const int j = v - p.seg[s].v0;
        if (p.seg[s].w2) {
            const void *w = j & 1 ? p.seg[s].w2 : p.seg[s].w;
            return static_cast<const T *>(w) + (size_t)(j >> 1) * p.pitch;
        }
        return j < p.seg[s].n ? static_cast<const T *>(p.seg[s].w) + (size_t)j * p.pitch : nullptr;
    };
    // Weights are never written: the first rows can be on their way to the L2 before the input exists.
    if (tid < p.prefetch && v_lo + tid < v_hi) {
        const T *w = weight_row(find(v_lo + tid), v_lo + tid);
        if (w) prefetch_l2(w, (uint32_t)(row_floats * sizeof(T)));
    }
    int need = p.h_out && blockIdx.x == 0 ? 2 : 0;  // bit i: this CTA's rows read normalized input i
    if (v_lo < v_hi)
        for (int s = find(v_lo); s < p.n_seg && p.seg[s].v0 < v_hi; s++) need |= 1 << p.seg[s].input;
    if (!p.xn)
#pragma unroll 4
        for (int c = tid; c < 2 * pieces; c += kThreads) {
            const int o = c >= pieces;
            if (need >> o & 1) nw[c] = __ldg(static_cast<const uint4 *>(p.norm_w[o]) + (c - o * pieces));
        }
    pdl_enter();

    constexpr int N = Vec<T>::N;
    if (p.xn) {
#pragma unroll 4
        for (int c = tid; c < pieces; c += kThreads) {
            float f[N];
            unpack(__ldcg(static_cast<const uint4 *>(p.xn) + c), f);
            cut_piece<T>(c, p.k, f);
            put_piece<T>(xs[0], c, pieces, f);
        }
    } else {
        float s = 0.f;
#pragma unroll 2
        for (int c = tid; c < pieces; c += kThreads) {
            float f[N];
            load_f32_piece<T>(p.x, c, p.k, f);
            put_piece<T>(xs[1], c, pieces, f);
#pragma unroll
            for (int j = 0; j < N; j++) s += f[j];
        }
        const float mean = block_sum(s, red) / (float)p.k;
        float q = 0.f;
        for (int c = tid; c < pieces; c += kThreads) {
            float f[N];
            get_piece<T>(xs[1], c, pieces, f);
#pragma unroll
            for (int j = 0; j < N; j++) q += N * c + j < p.k ? (f[j] - mean) * (f[j] - mean) : 0.f;
        }
        const float rstd = 1.0f / sqrtf(block_sum(q, red) / (float)p.k + p.eps);
        for (int c = tid; c < pieces; c += kThreads) {
            float f[N], w[N], h[N];
            get_piece<T>(xs[1], c, pieces, f);
#pragma unroll
            for (int o = 0; o < 2; o++) {
                if (!(need >> o & 1)) continue;
                unpack(nw[o * pieces + c], w);  // padded with zeros
#pragma unroll
                for (int j = 0; j < N; j++) h[j] = (f[j] - mean) * rstd * w[j];
                put_piece<T>(xs[o], c, pieces, h);
            }
            if (p.h_out && blockIdx.x == 0)
#pragma unroll
                for (int j = 0; j < N; j++)
                    if (N * c + j < p.k) p.h_out[N * c + j] = h[j];
        }
    }
    __syncthreads();

    const int rows = v_hi - v_lo, per = (pieces + p.split - 1) / p.split;
    stream_items<T, kWarps>(rows, p.split, smem, smem + 4 * pieces, part, [&](int r, int t) {
        Item it;
        const int s = find(v_lo + r);
        const T *w = weight_row(s, v_lo + r);
        share_of(per, pieces, t, it);
        if (!w) it.hi = it.lo;
        it.w = reinterpret_cast<const uint4 *>(w);
        it.shift = p.seg[s].input ? pieces * (Vec<T>::N / 4) : 0;  // the second input lies behind the first
        it.slot = r * p.split + t;
        it.scale = 1.f;
        return it;
    });
    __syncthreads();
    auto total = [&](int r) {
        float a = 0.f;
        for (int i = 0; i < p.split; i++) a += part[r * p.split + i];
        return a;
    };
    for (int r = tid; r < rows; r += kThreads) {
        const int v = v_lo + r, s = find(v);
        const GemvSeg &g = p.seg[s];
        const int j = v - g.v0;
        if (g.w2) {
            if (j & 1) continue;
            float gate = total(r), up = total(r + 1);
            if (g.bias) gate += to_f32(static_cast<const T *>(g.bias)[j >> 1]);
            if (g.bias2) up += to_f32(static_cast<const T *>(g.bias2)[j >> 1]);
            static_cast<T *>(g.out)[j >> 1] =
                from_f32<T>(g.epi == EPI_CLAMPED_GLU ? clamped_glu(gate, up, g.limit) : silu_mul(gate, up));
        } else if (j < g.n) {
            float a = total(r);
            if (g.bias) a += to_f32(static_cast<const T *>(g.bias)[j]);
            if (g.epi == EPI_SOFTCAP_F32) a = g.limit * tanhf(a / g.limit);
            if (g.epi == EPI_STORE_F32 || g.epi == EPI_SOFTCAP_F32)
                static_cast<float *>(g.out)[j] = a;
            else
                static_cast<T *>(g.out)[j] = from_f32<T>(a);
        }
    }
}

// The `top` largest sigmoid scores of `experts` logits (the lowest index of equals first).  One
// warp; `score` holds `experts` floats and is consumed.
__device__ __forceinline__ void choose_experts(const float *logits, int experts, int top, float *score, int *chosen,
                                               float *weight, int lane) {
    for (int e = lane; e < experts; e += 32) score[e] = sigmoid_f(__ldcg(logits + e));
    __syncwarp();
    for (int t = 0; t < top; t++) {
        float best = -1.f;
        int bi = experts;
        for (int e = lane; e < experts; e += 32)
            if (score[e] > best) {
                best = score[e];
                bi = e;
            }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > best || (ov == best && oi < bi)) {
                best = ov;
                bi = oi;
            }
        }
        if (bi >= experts) bi = 0;  // scores that are not numbers: stay inside the tables
        if (lane == 0) {
            chosen[t] = bi;
            weight[t] = best;
            score[bi] = -2.f;
        }
        __syncwarp();
    }
}

// Runs beside the attention of its layer: launched after it, it may be scheduled as soon as every
// attention CTA has passed its own dependency wait, when the kernel before the attention -- the
// writer of everything read here -- is complete.  It waits for the attention only before it ends,
// so that whoever waits for this kernel has waited for both.
template <typename T>
__global__ void __launch_bounds__(kThreads, 2) expert_gemv_kernel(const __grid_constant__ ExpertParams p) {
    extern __shared__ __align__(16) float smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pieces = (p.k + Vec<T>::N - 1) / Vec<T>::N;
    const int row_floats = pieces * Vec<T>::N;
    float *xs = smem, *part = smem + row_floats;
    float *score = part + (size_t)p.rows_cap * p.split;
    float *weight = score + p.experts;
    int *chosen = reinterpret_cast<int *>(weight + p.top);
    const void **tab = reinterpret_cast<const void **>((reinterpret_cast<uintptr_t>(chosen + p.top) + 7) & ~(uintptr_t)7);  // [top][gate, up]
    pdl_trigger();

    if (warp == 0) {
        choose_experts(p.logits, p.experts, p.top, score, chosen, weight, lane);
        for (int t = lane; t < p.top; t += 32) {
            tab[2 * t] = p.gate[chosen[t]];
            tab[2 * t + 1] = p.up[chosen[t]];
        }
    } else {
#pragma unroll 2
        for (int c = tid - 32; c < pieces; c += kThreads - 32) {
            float f[Vec<T>::N];
            load_f32_piece<T>(p.h, c, p.k, f);
            put_piece<T>(xs, c, pieces, f);
        }
    }
    __syncthreads();
    if (blockIdx.x == 0 && tid < p.top) {
        p.chosen[tid] = chosen[tid];
        p.weight[tid] = weight[tid];
    }
    // virtual rows: [choice][output][gate, up]
    const int pairs = p.top * p.ff;
    const int u_lo = (int)((long long)pairs * blockIdx.x / gridDim.x);
    const int u_hi = (int)((long long)pairs * (blockIdx.x + 1) / gridDim.x);
    const int per = (pieces + p.split - 1) / p.split;
    stream_items<T, kWarps>(2 * (u_hi - u_lo), p.split, xs, xs + 4 * pieces, part, [&](int r, int t) {
        Item it;
        const int u = u_lo + (r >> 1), c = u / p.ff;
        const void *w = tab[2 * c + (r & 1)];
        share_of(per, pieces, t, it);
        it.w = reinterpret_cast<const uint4 *>(static_cast<const T *>(w) + (size_t)(u - c * p.ff) * p.pitch);
        it.shift = 0;
        it.slot = r * p.split + t;
        it.scale = 1.f;
        return it;
    });
    __syncthreads();
    for (int u = u_lo + tid; u < u_hi; u += kThreads) {
        const int c = u / p.ff, j = u - c * p.ff, r = 2 * (u - u_lo);
        float gate = 0.f, up = 0.f;
        for (int i = 0; i < p.split; i++) {
            gate += part[r * p.split + i];
            up += part[(r + 1) * p.split + i];
        }
        static_cast<T *>(p.act)[(size_t)c * p.act_pitch + j] = from_f32<T>(silu_mul(weight[c] * gate, weight[c] * up));
    }
    pdl_wait();
}

template <typename T>
__global__ void __launch_bounds__(kThreads, 2) out_gemv_kernel(const __grid_constant__ OutParams p) {
    extern __shared__ __align__(16) float smem[];
    const int tid = threadIdx.x;
    float *part = smem + (size_t)p.pieces * Vec<T>::N;
    const int slots = p.seg[0].split + (p.n_seg > 1 ? p.seg[1].split : 0) + p.top * p.expert_split;
    const void **down = reinterpret_cast<const void **>(part + (((size_t)p.rows_cap * slots + 1) & ~(size_t)1));
    const int r_lo = (int)((long long)p.n * blockIdx.x / gridDim.x);
    const int r_hi = (int)((long long)p.n * (blockIdx.x + 1) / gridDim.x);
    for (int s = 0; s < p.n_seg; s++)
        if (tid < p.prefetch && r_lo + tid < r_hi)
            prefetch_l2(static_cast<const T *>(p.seg[s].w) + (size_t)(r_lo + tid) * p.seg[s].pitch,
                        (uint32_t)(((p.seg[s].k * (int)sizeof(T)) + 15) & ~15));
    pdl_enter();
    const int n_dense = p.expert_c0;
#pragma unroll 4
    for (int c = tid; c < p.pieces; c += kThreads) {
        const T *in;
        int at, k;
        if (c < n_dense) {
            const int s = p.n_seg > 1 && c >= p.seg[1].c0 ? 1 : 0;
            in = static_cast<const T *>(p.seg[s].in);
            at = c - p.seg[s].c0;
            k = p.seg[s].k;
        } else {
            const int e = (c - n_dense) / p.expert_pieces;
            in = static_cast<const T *>(p.expert_in) + (size_t)e * p.expert_in_pitch;
            at = c - n_dense - e * p.expert_pieces;
            k = p.expert_k;
        }
        float f[Vec<T>::N];
        unpack(__ldcg(reinterpret_cast<const uint4 *>(in) + at), f);
        cut_piece<T>(at, k, f);
        put_piece<T>(smem, c, p.pieces, f);
    }
    float seg_scale[2] = {1.f, 1.f};
    for (int s = 0; s < p.n_seg; s++)
        if (p.seg[s].scale_logit) seg_scale[s] = sigmoid_f(__ldcg(p.seg[s].scale_logit));
    if (tid < p.top) down[tid] = p.down[__ldcg(p.chosen + tid)];
    __syncthreads();
    const int rows = r_hi - r_lo;
    const int split0 = p.seg[0].split, split1 = p.n_seg > 1 ? p.seg[1].split : 0;
    const int pieces0 = (p.seg[0].k + Vec<T>::N - 1) / Vec<T>::N, per0 = (pieces0 + split0 - 1) / split0;
    const int pieces1 = split1 ? (p.seg[1].k + Vec<T>::N - 1) / Vec<T>::N : 0, per1 = split1 ? (pieces1 + split1 - 1) / split1 : 1;
    const int per_e = (p.expert_pieces + p.expert_split - 1) / p.expert_split;
    stream_items<T, kWarps>(rows, slots, smem, smem + 4 * (size_t)p.pieces, part, [&](int r, int t) {
        Item it;
        it.slot = r * slots + t;
        it.scale = 1.f;
        if (t < split0) {
            share_of(per0, pieces0, t, it);
            it.w = reinterpret_cast<const uint4 *>(static_cast<const T *>(p.seg[0].w) + (size_t)(r_lo + r) * p.seg[0].pitch);
            it.shift = 0;
            it.scale = seg_scale[0];
        } else if (t < split0 + split1) {
            share_of(per1, pieces1, t - split0, it);
            it.w = reinterpret_cast<const uint4 *>(static_cast<const T *>(p.seg[1].w) + (size_t)(r_lo + r) * p.seg[1].pitch);
            it.shift = p.seg[1].c0;
            it.scale = seg_scale[1];
        } else {
            t -= split0 + split1;
            const int c = p.expert_split == 1 ? t : t / p.expert_split;
            share_of(per_e, p.expert_pieces, t - c * p.expert_split, it);
            it.w = reinterpret_cast<const uint4 *>(static_cast<const T *>(down[c]) + (size_t)(r_lo + r) * p.expert_pitch);
            it.shift = p.expert_c0 + c * p.expert_pieces;
        }
        return it;
    });
    __syncthreads();
    for (int r = tid; r < rows; r += kThreads) {
        float a = 0.f;
        for (int i = 0; i < slots; i++) a += part[r * slots + i];
        const int n = r_lo + r;
        if (p.bias) a += to_f32(static_cast<const T *>(p.bias)[n]);
        if (p.st.n > 0)
            streams_column<T>(p.st, 0, p.n, n, a);
        else
            p.x[n] = __ldcg(p.x + n) + a;
    }
}

// Grid and stretches per row for `units` of `rows_per_unit` weight rows of `pieces` 16-byte pieces:
// up to two CTAs per SM (one when the inputs fill the shared memory), and the split that spreads the
// rows most evenly over the warps at the least bookkeeping.
struct Shape {
    int grid, split, rows_cap;
};
int grid_for(const tlc_ctx *ctx, int units, long items, size_t input_bytes) {
    int grid = (input_bytes > 96 * 1024 ? 1 : 2) * ctx->sm_count;
    const long want = (items + kWarps - 1) / kWarps;
    if (want < grid) grid = (int)want;
    if (grid > units) grid = units;
    return grid < 1 ? 1 : grid;
}
Shape choose_shape(const tlc_ctx *ctx, int units, int rows_per_unit, int pieces, size_t input_bytes) {
    Shape best{1, 1, 0};
    double best_cost = 1e30;
    for (int split = 1; split <= 16; split *= 2) {
        if (split > 1 && pieces / split < 32) break;
        const int grid = grid_for(ctx, units, (long)units * rows_per_unit * split, input_bytes);
        const int cap = (units + grid - 1) / grid * rows_per_unit;
        const int per_warp = (cap * split + kWarps - 1) / kWarps;
        const double batches = (double)(((pieces + split - 1) / split + 32 * kBatch - 1) / (32 * kBatch));
        const double cost = per_warp * (batches + 0.5);  // an item's reduction costs about half a batch
        if (cost < best_cost * 0.98) {
            best_cost = cost;
            best = {grid, split, cap};
        }
    }
    return best;
}
// Stretches of a segment of `pieces` in the output kernel: two batches of a lane each.
int split_for(int pieces) { return pieces <= 256 ? 1 : (pieces + 255) / 256; }

template <typename K>
int32_t set_limits(K kernel, bool (&done)[64], int device) {
    if (done[device & 63]) return TLC_OK;
    TLC_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(kSmemMax + 16 * 1024)));
    TLC_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared));
    done[device & 63] = true;
    return TLC_OK;
}

}  // namespace

bool gemv_fits(int k) { return (size_t)4 * (k + 8) * sizeof(float) <= kSmemMax; }

#define TLC_LAUNCHED(ctx, le, what)                                                            \
    do {                                                                                       \
        if ((le) != cudaSuccess) {                                                             \
            cudaGetLastError();                                                                \
            return tlc_fail(TLC_ERR_CUDA, what " launch failed: %s", cudaGetErrorString(le));  \
        }                                                                                      \
        TLC_CHECK_LAUNCH(ctx);                                                                 \
    } while (0)

template <typename T>
int32_t launch_gemv(tlc_ctx *ctx, GemvParams &p) {
    static bool done[64] = {};
    if (int32_t rc = set_limits(gemv_kernel<T>, done, ctx->device)) return rc;
    int v = 0;
    for (int s = 0; s < p.n_seg; s++) {
        p.seg[s].v0 = v;
        v += p.seg[s].w2 ? 2 * p.seg[s].n : (p.seg[s].n + 1) & ~1;
    }
    p.v_total = v;
    const int pieces = (p.k + Vec<T>::N - 1) / Vec<T>::N;
    const size_t input = (size_t)2 * pieces * 16 / sizeof(T) * sizeof(float) + (p.xn ? 0 : (size_t)2 * pieces * 16);
    const Shape sh = choose_shape(ctx, v / 2, 2, pieces, input);
    p.split = sh.split;
    p.rows_cap = sh.rows_cap;
    const size_t smem = input + (size_t)sh.rows_cap * sh.split * sizeof(float);
    TLC_REQUIRE(smem <= kSmemMax + 16 * 1024, TLC_ERR_INVALID_OPERATION, "dense gemv: %d inputs do not fit the shared memory", p.k);
    p.prefetch = (int)(96 * 1024 / ((size_t)pieces * 16));
    cudaError_t le = tlc_launch_pdl(ctx, gemv_kernel<T>, dim3(sh.grid), dim3(kThreads), smem, p);
    TLC_LAUNCHED(ctx, le, "dense gemv");
    return TLC_OK;
}

// Shapes of the two launches below and the shared memory they take.
template <typename T>
static size_t plan_expert(const tlc_ctx *ctx, ExpertParams &p, int *grid) {
    const int pieces = (p.k + Vec<T>::N - 1) / Vec<T>::N;
    const size_t input = (size_t)pieces * 16 / sizeof(T) * sizeof(float);
    const Shape sh = choose_shape(ctx, p.top * p.ff, 2, pieces, input);
    p.split = sh.split;
    p.rows_cap = sh.rows_cap;
    *grid = sh.grid;
    return input + (size_t)sh.rows_cap * sh.split * sizeof(float) + ((size_t)p.experts + 2 * p.top) * 4 + (size_t)2 * p.top * sizeof(void *) + 8;
}
template <typename T>
static size_t plan_out(const tlc_ctx *ctx, OutParams &p, int *grid) {
    int c = 0, slots = 0;
    int64_t dense_bytes = 0;
    for (int s = 0; s < p.n_seg; s++) {
        const int pieces = (p.seg[s].k + Vec<T>::N - 1) / Vec<T>::N;
        p.seg[s].c0 = c;
        p.seg[s].split = split_for(pieces);
        c += pieces;
        slots += p.seg[s].split;
        dense_bytes += (int64_t)pieces * 16;
    }
    p.expert_c0 = c;
    p.expert_pieces = (p.expert_k + Vec<T>::N - 1) / Vec<T>::N;
    p.expert_split = p.top ? split_for(p.expert_pieces) : 1;
    p.pieces = c + p.top * p.expert_pieces;
    slots += p.top * p.expert_split;
    const size_t input = (size_t)p.pieces * Vec<T>::N * sizeof(float);
    *grid = grid_for(ctx, p.n, (long)p.n * slots, input);
    p.rows_cap = (p.n + *grid - 1) / *grid;
    p.prefetch = dense_bytes ? (int)(128 * 1024 / dense_bytes) : 0;
    return input + ((size_t)p.rows_cap * slots + 1) * sizeof(float) + (size_t)p.top * sizeof(void *) + 8;
}

template <typename T>
bool layer_gemv_fits(const tlc_ctx *ctx, ExpertParams e, OutParams o) {
    int grid;
    if (e.top > 0 && (e.top > kThreads || plan_expert<T>(ctx, e, &grid) > kSmemMax + 16 * 1024)) return false;
    return plan_out<T>(ctx, o, &grid) <= kSmemMax + 16 * 1024;
}

template <typename T>
int32_t launch_expert_gemv(tlc_ctx *ctx, ExpertParams &p) {
    static bool done[64] = {};
    if (int32_t rc = set_limits(expert_gemv_kernel<T>, done, ctx->device)) return rc;
    int grid = 1;
    const size_t smem = plan_expert<T>(ctx, p, &grid);
    TLC_REQUIRE(smem <= kSmemMax + 16 * 1024 && p.top <= kThreads, TLC_ERR_INVALID_OPERATION,
                "expert gemv: %d inputs do not fit the shared memory", p.k);
    cudaError_t le = tlc_launch_pdl(ctx, expert_gemv_kernel<T>, dim3(grid), dim3(kThreads), smem, p);
    TLC_LAUNCHED(ctx, le, "expert gemv");
    return TLC_OK;
}

template <typename T>
int32_t launch_out_gemv(tlc_ctx *ctx, OutParams &p) {
    static bool done[64] = {};
    if (int32_t rc = set_limits(out_gemv_kernel<T>, done, ctx->device)) return rc;
    int grid = 1;
    const size_t smem = plan_out<T>(ctx, p, &grid);
    TLC_REQUIRE(smem <= kSmemMax + 16 * 1024 && p.top <= kThreads, TLC_ERR_INVALID_OPERATION,
                "output gemv: %d inputs do not fit the shared memory", p.pieces * Vec<T>::N);
    cudaError_t le = tlc_launch_pdl(ctx, out_gemv_kernel<T>, dim3(grid), dim3(kThreads), smem, p);
    TLC_LAUNCHED(ctx, le, "output gemv");
    return TLC_OK;
}

template bool layer_gemv_fits<bf16>(const tlc_ctx *, ExpertParams, OutParams);
template bool layer_gemv_fits<float>(const tlc_ctx *, ExpertParams, OutParams);
template int32_t launch_gemv<bf16>(tlc_ctx *, GemvParams &);
template int32_t launch_gemv<float>(tlc_ctx *, GemvParams &);
template int32_t launch_expert_gemv<bf16>(tlc_ctx *, ExpertParams &);
template int32_t launch_expert_gemv<float>(tlc_ctx *, ExpertParams &);
template int32_t launch_out_gemv<bf16>(tlc_ctx *, OutParams &);
template int32_t launch_out_gemv<float>(tlc_ctx *, OutParams &);

}  // namespace tlc_dense
