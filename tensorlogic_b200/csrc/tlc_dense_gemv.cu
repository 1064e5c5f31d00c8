// One activation row against dense weights: the decode step of one sequence.
//
// Three kernels, one launch each:
//   gemv_kernel         layer norm(s) of the residual row, then several weights against the
//                       normalized inputs (q, k, gate/up pairs, router, lm_head);
//   expert_gemv_kernel  router decision, then gate/up of the chosen experts;
//   out_gemv_kernel     the projections back into the residual stream -- attention output,
//                       feed-forward down, chosen experts, shared expert -- as ONE sum per output.
// All are bound by the weights' bytes.  A warp streams a weight row, or 1 / 2^s of one, in 16-byte
// loads; CTAs own contiguous rows, the partial sums meet in shared memory after the last load, so
// no barrier interrupts the stream.  The input sits in shared memory as f32, unrounded.
#include <cstring>

#include "tlc_dense.cuh"

namespace tlc_dense {

namespace {

constexpr int kThreads = 512, kWarps = kThreads / 32;
constexpr int kUnroll = 8;  // 16-byte loads in flight per lane
constexpr size_t kSmemMax = 200 * 1024;

// Input layout in shared memory: piece c (16 bytes of weights) faces floats 4 c .. 4 c + 3 of plane
// 0 and, for bf16, of plane 1, so that a warp's 16-byte reads fall on distinct banks.
template <typename T>
__device__ __forceinline__ int plane_index(int i, int pieces) {
    if (Vec<T>::N == 4) return i;
    return (i >> 3) * 4 + (i & 3) + ((i >> 2) & 1) * pieces * 4;
}

__device__ __forceinline__ uint4 load_weight(const uint4 *p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];"
                 : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
                 : "l"(p));
    return v;
}
__device__ __forceinline__ void prefetch_l2(const void *p, uint32_t bytes) {
    asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(p), "r"(bytes) : "memory");
}

template <typename T>
__device__ __forceinline__ float dot_piece(const uint4 &w, const float *plane0, const float *plane1, int c) {
    float f[Vec<T>::N];
    unpack(w, f);
    const float4 a = *reinterpret_cast<const float4 *>(plane0 + 4 * c);
    float s = f[0] * a.x;
    s = fmaf(f[1], a.y, s);
    s = fmaf(f[2], a.z, s);
    s = fmaf(f[3], a.w, s);
    if constexpr (Vec<T>::N == 8) {
        const float4 b = *reinterpret_cast<const float4 *>(plane1 + 4 * c);
        s = fmaf(f[4], b.x, s);
        s = fmaf(f[5], b.y, s);
        s = fmaf(f[6], b.z, s);
        s = fmaf(f[7], b.w, s);
    }
    return s;
}

// This lane's share of pieces [c_lo, c_hi) of a weight row against the input pieces of the same
// numbers shifted by `shift`.
template <typename T>
__device__ __forceinline__ float dot_row(const uint4 *row, const float *plane0, const float *plane1, int c_lo, int c_hi,
                                         int shift, int lane) {
    float s = 0.f;
    for (int c = c_lo + lane; c < c_hi; c += 32 * kUnroll) {
        uint4 w[kUnroll];
#pragma unroll
        for (int u = 0; u < kUnroll; u++)
            w[u] = c + 32 * u < c_hi ? load_weight(row + c + 32 * u) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
        for (int u = 0; u < kUnroll; u++)
            if (c + 32 * u < c_hi) s += dot_piece<T>(w[u], plane0, plane1, c + 32 * u + shift);
    }
    return s;
}

struct Share {  // pieces of a row warp `part` of 2^log2 takes
    int lo, hi;
};
__device__ __forceinline__ Share share_of(int pieces, int part, int log2) {
    const int per = (pieces + (1 << log2) - 1) >> log2;
    const int lo = part * per;
    return {lo < pieces ? lo : pieces, lo + per < pieces ? lo + per : pieces};
}

template <typename T>
__global__ void __launch_bounds__(kThreads, 2) gemv_kernel(const __grid_constant__ GemvParams p) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float red[33];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pieces = (p.k + Vec<T>::N - 1) / Vec<T>::N;
    const int row_floats = pieces * Vec<T>::N;
    float *xs[2] = {smem, smem + row_floats};
    float *part = smem + 2 * (size_t)row_floats;

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
    bool need[2] = {false, p.h_out != nullptr && blockIdx.x == 0};
    if (v_lo < v_hi)
        for (int s = find(v_lo); s < p.n_seg && p.seg[s].v0 < v_hi; s++) need[p.seg[s].input] = true;
    pdl_enter();

    if (p.xn) {
        const T *x = static_cast<const T *>(p.xn);
        for (int i = tid; i < row_floats; i += kThreads) xs[0][plane_index<T>(i, pieces)] = i < p.k ? to_f32(x[i]) : 0.f;
    } else {
        float s = 0.f;
        for (int i = tid; i < row_floats; i += kThreads) {
            const float v = i < p.k ? __ldcg(p.x + i) : 0.f;
            xs[1][plane_index<T>(i, pieces)] = v;
            s += v;
        }
        const float mean = block_sum(s, red) / (float)p.k;
        float q = 0.f;
        for (int i = tid; i < p.k; i += kThreads) {
            const float dlt = xs[1][plane_index<T>(i, pieces)] - mean;
            q += dlt * dlt;
        }
        const float rstd = 1.0f / sqrtf(block_sum(q, red) / (float)p.k + p.eps);
        const T *w0 = static_cast<const T *>(p.norm_w[0]), *w1 = static_cast<const T *>(p.norm_w[1]);
        for (int i = tid; i < p.k; i += kThreads) {
            const int at = plane_index<T>(i, pieces);
            const float xh = (xs[1][at] - mean) * rstd;
            if (need[0]) xs[0][at] = xh * to_f32(w0[i]);
            if (need[1]) {
                const float h = xh * to_f32(w1[i]);
                xs[1][at] = h;
                if (p.h_out && blockIdx.x == 0) p.h_out[i] = h;
            }
        }
        if (need[0])
            for (int i = p.k + tid; i < row_floats; i += kThreads) xs[0][plane_index<T>(i, pieces)] = 0.f;
    }
    __syncthreads();

    const int rows = v_hi - v_lo, ks = 1 << p.ksplit_log2;
    for (int it = warp; it < rows << p.ksplit_log2; it += kWarps) {
        const int r = it >> p.ksplit_log2, pt = it & (ks - 1);
        const int s = find(v_lo + r);
        const T *w = weight_row(s, v_lo + r);
        float acc = 0.f;
        if (w) {
            const Share sh = share_of(pieces, pt, p.ksplit_log2);
            const float *in = xs[p.seg[s].input];
            acc = dot_row<T>(reinterpret_cast<const uint4 *>(w), in, in + 4 * pieces, sh.lo, sh.hi, 0, lane);
            acc = warp_sum(acc);
        }
        if (lane == 0) part[it] = acc;
    }
    __syncthreads();
    auto total = [&](int r) {
        float a = 0.f;
        for (int i = 0; i < ks; i++) a += part[(r << p.ksplit_log2) + i];
        return a;
    };
    for (int r = tid; r < rows; r += kThreads) {
        const int v = v_lo + r, s = find(v);
        const GemvSeg &g = p.seg[s];
        const int j = v - g.v0;
        if (g.w2) {
            if (j & 1) continue;
            const float gate = total(r), up = total(r + 1);
            static_cast<T *>(g.out)[j >> 1] =
                from_f32<T>(g.epi == EPI_CLAMPED_GLU ? clamped_glu(gate, up, g.limit) : silu_mul(gate, up));
        } else if (j < g.n) {
            float a = total(r);
            if (g.bias) a += to_f32(static_cast<const T *>(g.bias)[j]);
            if (g.epi == EPI_STORE_F32)
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
__global__ void __launch_bounds__(kThreads, 2) expert_gemv_kernel(const __grid_constant__ ExpertParams p, int wait_first) {
    extern __shared__ __align__(16) float smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pieces = (p.k + Vec<T>::N - 1) / Vec<T>::N;
    const int row_floats = pieces * Vec<T>::N;
    float *xs = smem, *part = smem + row_floats;
    float *score = part + ((size_t)p.rows_cap << p.ksplit_log2);
    float *weight = score + p.experts;
    int *chosen = reinterpret_cast<int *>(weight + p.top);
    if (wait_first) pdl_wait();
    pdl_trigger();

    if (warp == 0) choose_experts(p.logits, p.experts, p.top, score, chosen, weight, lane);
    for (int i = tid; i < row_floats; i += kThreads) xs[plane_index<T>(i, pieces)] = i < p.k ? __ldcg(p.h + i) : 0.f;
    __syncthreads();
    if (blockIdx.x == 0 && tid < p.top) {
        p.chosen[tid] = chosen[tid];
        p.weight[tid] = weight[tid];
    }
    // virtual rows: [choice][output][gate, up]
    const int pairs = p.top * p.ff;
    const int u_lo = (int)((long long)pairs * blockIdx.x / gridDim.x);
    const int u_hi = (int)((long long)pairs * (blockIdx.x + 1) / gridDim.x);
    const int rows = 2 * (u_hi - u_lo), ks = 1 << p.ksplit_log2;
    for (int it = warp; it < rows << p.ksplit_log2; it += kWarps) {
        const int r = it >> p.ksplit_log2, pt = it & (ks - 1);
        const int u = u_lo + (r >> 1), c = u / p.ff, j = u - c * p.ff;
        const void *w = r & 1 ? p.up[chosen[c]] : p.gate[chosen[c]];
        const Share sh = share_of(pieces, pt, p.ksplit_log2);
        float acc = dot_row<T>(reinterpret_cast<const uint4 *>(static_cast<const T *>(w) + (size_t)j * p.pitch), xs,
                               xs + 4 * pieces, sh.lo, sh.hi, 0, lane);
        acc = warp_sum(acc);
        if (lane == 0) part[it] = acc;
    }
    __syncthreads();
    for (int u = u_lo + tid; u < u_hi; u += kThreads) {
        const int c = u / p.ff, j = u - c * p.ff, r = 2 * (u - u_lo);
        float gate = 0.f, up = 0.f;
        for (int i = 0; i < ks; i++) {
            gate += part[(r << p.ksplit_log2) + i];
            up += part[((r + 1) << p.ksplit_log2) + i];
        }
        static_cast<T *>(p.act)[(size_t)c * p.act_pitch + j] = from_f32<T>(silu_mul(weight[c] * gate, weight[c] * up));
    }
    if (!wait_first) pdl_wait();
}

template <typename T>
__global__ void __launch_bounds__(kThreads, 2) out_gemv_kernel(const __grid_constant__ OutParams p) {
    extern __shared__ __align__(16) float smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float *part = smem + (size_t)p.pieces * Vec<T>::N;
    const int r_lo = (int)((long long)p.n * blockIdx.x / gridDim.x);
    const int r_hi = (int)((long long)p.n * (blockIdx.x + 1) / gridDim.x);
    for (int s = 0; s < p.n_seg; s++)
        if (tid < p.prefetch && r_lo + tid < r_hi)
            prefetch_l2(static_cast<const T *>(p.seg[s].w) + (size_t)(r_lo + tid) * p.seg[s].pitch,
                        (uint32_t)(((p.seg[s].k * (int)sizeof(T)) + 15) & ~15));
    pdl_enter();
    float seg_scale[2] = {1.f, 1.f};
    for (int s = 0; s < p.n_seg; s++) {
        const T *in = static_cast<const T *>(p.seg[s].in);
        const int n = (p.seg[s].k + Vec<T>::N - 1) / Vec<T>::N * Vec<T>::N, base = p.seg[s].c0 * Vec<T>::N;
        for (int i = tid; i < n; i += kThreads)
            smem[plane_index<T>(base + i, p.pieces)] = i < p.seg[s].k ? to_f32(__ldcg(in + i)) : 0.f;
        if (p.seg[s].scale_logit) seg_scale[s] = sigmoid_f(__ldcg(p.seg[s].scale_logit));
    }
    for (int c = 0; c < p.top; c++) {
        const T *in = static_cast<const T *>(p.expert_in) + (size_t)c * p.expert_in_pitch;
        const int n = p.expert_pieces * Vec<T>::N, base = (p.expert_c0 + c * p.expert_pieces) * Vec<T>::N;
        for (int i = tid; i < n; i += kThreads)
            smem[plane_index<T>(base + i, p.pieces)] = i < p.expert_k ? to_f32(__ldcg(in + i)) : 0.f;
    }
    __syncthreads();
    const float *plane1 = smem + 4 * (size_t)p.pieces;
    const int rows = r_hi - r_lo, ks = 1 << p.ksplit_log2;
    for (int it = warp; it < rows << p.ksplit_log2; it += kWarps) {
        const int n = r_lo + (it >> p.ksplit_log2);
        const Share sh = share_of(p.pieces, it & (ks - 1), p.ksplit_log2);
        float acc = 0.f;
        for (int s = 0; s < p.n_seg; s++) {
            const int c0 = p.seg[s].c0, c1 = c0 + (p.seg[s].k + Vec<T>::N - 1) / Vec<T>::N;
            const int lo = sh.lo > c0 ? sh.lo : c0, hi = sh.hi < c1 ? sh.hi : c1;
            if (lo >= hi) continue;
            acc += seg_scale[s] * dot_row<T>(reinterpret_cast<const uint4 *>(static_cast<const T *>(p.seg[s].w) +
                                                                             (size_t)n * p.seg[s].pitch),
                                             smem, plane1, lo - c0, hi - c0, c0, lane);
        }
        for (int c = 0; c < p.top; c++) {
            const int c0 = p.expert_c0 + c * p.expert_pieces, c1 = c0 + p.expert_pieces;
            const int lo = sh.lo > c0 ? sh.lo : c0, hi = sh.hi < c1 ? sh.hi : c1;
            if (lo >= hi) continue;
            const T *w = static_cast<const T *>(p.down[__ldcg(p.chosen + c)]) + (size_t)n * p.expert_pitch;
            acc += dot_row<T>(reinterpret_cast<const uint4 *>(w), smem, plane1, lo - c0, hi - c0, c0, lane);
        }
        acc = warp_sum(acc);
        if (lane == 0) part[it] = acc;
    }
    __syncthreads();
    for (int r = tid; r < rows; r += kThreads) {
        float a = 0.f;
        for (int i = 0; i < ks; i++) a += part[(r << p.ksplit_log2) + i];
        const int n = r_lo + r;
        if (p.bias) a += to_f32(static_cast<const T *>(p.bias)[n]);
        p.x[n] = __ldcg(p.x + n) + a;
    }
}

// Grid and warps per row for `rows` weight rows of `pieces` 16-byte pieces: up to two CTAs per SM
// (one when the inputs fill the shared memory), and the smallest split that spreads the rows
// evenly over the warps without leaving a warp less than one full round of loads.
struct Shape {
    int grid, log2, rows_cap;
};
Shape choose_shape(const tlc_ctx *ctx, int units, int rows_per_unit, int pieces, size_t input_bytes) {
    const int per_sm = input_bytes > 96 * 1024 ? 1 : 2;
    Shape best{1, 0, 0};
    double best_cost = 1e30;
    for (int log2 = 0; log2 <= 4; log2++) {
        if (log2 > 0 && (pieces >> log2) < 32) break;
        int grid = per_sm * ctx->sm_count;
        const long items = (long)units * rows_per_unit << log2;
        const long want = (items + kWarps - 1) / kWarps;
        if (want < grid) grid = (int)want;
        if (grid > units) grid = units;
        if (grid < 1) grid = 1;
        const int cap = (units + grid - 1) / grid * rows_per_unit;
        const int per_warp = ((cap << log2) + kWarps - 1) / kWarps;
        // loads a lane makes one after the other, plus the cost of reducing and storing an item
        const int rounds = (((pieces + (1 << log2) - 1) >> log2) + 32 * kUnroll - 1) / (32 * kUnroll);
        const double loads = (double)((pieces + (1 << log2) - 1) >> log2) / 32.0;
        const double cost = per_warp * (loads + 1.5 * rounds + 2.0);
        if (cost < best_cost * 0.98) {
            best_cost = cost;
            best = {grid, log2, cap};
        }
    }
    return best;
}

template <typename K>
int32_t set_limits(K kernel, bool (&done)[64], int device) {
    if (done[device & 63]) return TLC_OK;
    TLC_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(kSmemMax + 16 * 1024)));
    TLC_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared));
    done[device & 63] = true;
    return TLC_OK;
}

}  // namespace

bool gemv_fits(int k) { return (size_t)2 * (k + 8) * sizeof(float) <= kSmemMax; }
bool out_gemv_fits(int64_t k_total) { return (size_t)k_total * sizeof(float) <= kSmemMax; }

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
    const size_t input = (size_t)2 * pieces * 16 / sizeof(T) * sizeof(float);
    const Shape sh = choose_shape(ctx, v / 2, 2, pieces, input);
    p.ksplit_log2 = sh.log2;
    p.rows_cap = sh.rows_cap;
    const size_t smem = input + ((size_t)sh.rows_cap << sh.log2) * sizeof(float);
    TLC_REQUIRE(smem <= kSmemMax + 16 * 1024, TLC_ERR_INVALID_OPERATION, "dense gemv: %d inputs do not fit the shared memory", p.k);
    p.prefetch = (int)(96 * 1024 / ((size_t)pieces * 16));
    cudaError_t le = tlc_launch_pdl(ctx, gemv_kernel<T>, dim3(sh.grid), dim3(kThreads), smem, p);
    TLC_LAUNCHED(ctx, le, "dense gemv");
    return TLC_OK;
}

template <typename T>
int32_t launch_expert_gemv(tlc_ctx *ctx, ExpertParams &p) {
    static bool done[64] = {};
    if (int32_t rc = set_limits(expert_gemv_kernel<T>, done, ctx->device)) return rc;
    const int pieces = (p.k + Vec<T>::N - 1) / Vec<T>::N;
    const size_t input = (size_t)pieces * 16 / sizeof(T) * sizeof(float);
    const Shape sh = choose_shape(ctx, p.top * p.ff, 2, pieces, input);
    p.ksplit_log2 = sh.log2;
    p.rows_cap = sh.rows_cap;
    const size_t smem = input + ((size_t)sh.rows_cap << sh.log2) * sizeof(float) + ((size_t)p.experts + 2 * p.top) * 4;
    TLC_REQUIRE(smem <= kSmemMax + 16 * 1024 && p.top <= kThreads, TLC_ERR_INVALID_OPERATION,
                "expert gemv: %d inputs do not fit the shared memory", p.k);
    // Without dependent launch the kernels run one after the other anyway; the wait is then a no-op.
    cudaError_t le = tlc_launch_pdl(ctx, expert_gemv_kernel<T>, dim3(sh.grid), dim3(kThreads), smem, p, 0);
    TLC_LAUNCHED(ctx, le, "expert gemv");
    return TLC_OK;
}

template <typename T>
int32_t launch_out_gemv(tlc_ctx *ctx, OutParams &p) {
    static bool done[64] = {};
    if (int32_t rc = set_limits(out_gemv_kernel<T>, done, ctx->device)) return rc;
    int c = 0;
    int64_t dense_bytes = 0;
    for (int s = 0; s < p.n_seg; s++) {
        p.seg[s].c0 = c;
        const int pieces = (p.seg[s].k + Vec<T>::N - 1) / Vec<T>::N;
        c += pieces;
        dense_bytes += (int64_t)pieces * 16;
    }
    p.expert_c0 = c;
    p.expert_pieces = (p.expert_k + Vec<T>::N - 1) / Vec<T>::N;
    p.pieces = c + p.top * p.expert_pieces;
    const size_t input = (size_t)p.pieces * Vec<T>::N * sizeof(float);
    const Shape sh = choose_shape(ctx, p.n, 1, p.pieces, input);
    p.ksplit_log2 = sh.log2;
    p.rows_cap = sh.rows_cap;
    const size_t smem = input + ((size_t)sh.rows_cap << sh.log2) * sizeof(float);
    TLC_REQUIRE(smem <= kSmemMax + 16 * 1024, TLC_ERR_INVALID_OPERATION, "output gemv: %d inputs do not fit the shared memory",
                p.pieces * Vec<T>::N);
    p.prefetch = dense_bytes ? (int)(128 * 1024 / dense_bytes) : 0;
    cudaError_t le = tlc_launch_pdl(ctx, out_gemv_kernel<T>, dim3(sh.grid), dim3(kThreads), smem, p);
    TLC_LAUNCHED(ctx, le, "output gemv");
    return TLC_OK;
}

template int32_t launch_gemv<bf16>(tlc_ctx *, GemvParams &);
template int32_t launch_gemv<float>(tlc_ctx *, GemvParams &);
template int32_t launch_expert_gemv<bf16>(tlc_ctx *, ExpertParams &);
template int32_t launch_expert_gemv<float>(tlc_ctx *, ExpertParams &);
template int32_t launch_out_gemv<bf16>(tlc_ctx *, OutParams &);
template int32_t launch_out_gemv<float>(tlc_ctx *, OutParams &);

}  // namespace tlc_dense
