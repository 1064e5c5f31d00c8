// Row-wise steps of the config-driven decoder: embedding into the f32 residual stream, layer
// norms, query/key norm + rotation + cache append, expert choice and the permutation of rows by
// expert.
#include "tlc_dense.cuh"

namespace tlc_dense {

namespace {

// Four neighbouring values.
__device__ __forceinline__ void load4(const float *p, float (&f)[4]) {
    const float4 v = *reinterpret_cast<const float4 *>(p);
    f[0] = v.x;
    f[1] = v.y;
    f[2] = v.z;
    f[3] = v.w;
}
__device__ __forceinline__ void load4(const bf16 *p, float (&f)[4]) {
    const uint2 v = *reinterpret_cast<const uint2 *>(p);
    f[0] = __uint_as_float(v.x << 16);
    f[1] = __uint_as_float(v.x & 0xffff0000u);
    f[2] = __uint_as_float(v.y << 16);
    f[3] = __uint_as_float(v.y & 0xffff0000u);
}
__device__ __forceinline__ void store4(float *p, const float (&f)[4]) {
    *reinterpret_cast<float4 *>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
__device__ __forceinline__ void store4(bf16 *p, const float (&f)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
}

template <typename T>
__global__ void embed_rows_kernel(const T *__restrict__ table, int64_t pitch, int vocab, int d, const int *__restrict__ ids,
                                  float *__restrict__ x) {
    constexpr int N = Vec<T>::N;
    pdl_enter();  // ids are written by the previous step's sampling kernel
    const int r = blockIdx.y;
    int id = ids[r];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);  // ids are validated on the host; never read outside
    const T *src = table + (size_t)id * pitch;
    float *dst = x + (size_t)r * d;
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * N;
    if (i >= d) return;
    float f[N];
    unpack(__ldg(reinterpret_cast<const uint4 *>(src + i)), f);  // rows are padded to whole pieces
    if ((d & 3) == 0 && i + N <= d) {
#pragma unroll
        for (int e = 0; e < N; e += 4) *reinterpret_cast<float4 *>(dst + i + e) = make_float4(f[e], f[e + 1], f[e + 2], f[e + 3]);
    } else {
#pragma unroll
        for (int e = 0; e < N; e++)
            if (i + e < d) dst[i + e] = f[e];
    }
}

// One CTA per row.
template <typename T>
__global__ void __launch_bounds__(256) norm_rows_kernel(const NormParams p) {
    extern __shared__ float row[];
    __shared__ float red[33];
    pdl_enter();
    const int tid = threadIdx.x;
    if (p.zero)
        for (int i = blockIdx.x * blockDim.x + tid; i < p.n_zero; i += gridDim.x * blockDim.x) p.zero[i] = 0;
    const int src = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
    float *x = p.x + (size_t)src * p.d;
    if ((p.d & 3) == 0) {  // rows start on 16-byte boundaries
        float s = 0.f;
        for (int i = 4 * tid; i < p.d; i += 4 * blockDim.x) {
            float4 v = __ldcg(reinterpret_cast<const float4 *>(x + i));
            if (p.y) {
                float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
                for (int t = 0; t < p.top; t++) {
                    float f[4];
                    load4(static_cast<const T *>(p.y) + (size_t)p.place[(size_t)src * p.top + t] * p.y_pitch + i, f);
                    a.x += f[0];
                    a.y += f[1];
                    a.z += f[2];
                    a.w += f[3];
                }
                v.x += a.x;
                v.y += a.y;
                v.z += a.z;
                v.w += a.w;
                if (!p.rows) *reinterpret_cast<float4 *>(x + i) = v;
            }
            *reinterpret_cast<float4 *>(row + i) = v;
            s += (v.x + v.y) + (v.z + v.w);
        }
        const float mean = block_sum(s, red) / (float)p.d;
        float q = 0.f;
        for (int i = 4 * tid; i < p.d; i += 4 * blockDim.x) {
            const float4 v = *reinterpret_cast<const float4 *>(row + i);
            const float a = v.x - mean, b = v.y - mean, c = v.z - mean, e = v.w - mean;
            q += (a * a + b * b) + (c * c + e * e);
        }
        const float rstd = 1.0f / sqrtf(block_sum(q, red) / (float)p.d + p.eps);
        for (int i = 4 * tid; i < p.d; i += 4 * blockDim.x) {
            const float4 v = *reinterpret_cast<const float4 *>(row + i);
            const float h[4] = {(v.x - mean) * rstd, (v.y - mean) * rstd, (v.z - mean) * rstd, (v.w - mean) * rstd};
#pragma unroll
            for (int o = 0; o < 2; o++) {
                if (!p.w[o]) continue;
                float f[4];
                load4(static_cast<const T *>(p.w[o]) + i, f);
#pragma unroll
                for (int e = 0; e < 4; e++) f[e] *= h[e];
                store4(static_cast<T *>(p.out[o]) + (size_t)blockIdx.x * p.ldo + i, f);
            }
        }
        return;
    }
    float s = 0.f;
    for (int i = tid; i < p.d; i += blockDim.x) {
        float v = __ldcg(x + i);
        if (p.y) {
            float a = 0.f;
            for (int t = 0; t < p.top; t++)
                a += to_f32(static_cast<const T *>(p.y)[(size_t)p.place[(size_t)src * p.top + t] * p.y_pitch + i]);
            v += a;
            if (!p.rows) x[i] = v;
        }
        row[i] = v;
        s += v;
    }
    const float mean = block_sum(s, red) / (float)p.d;
    float q = 0.f;
    for (int i = tid; i < p.d; i += blockDim.x) {
        const float dlt = row[i] - mean;
        q += dlt * dlt;
    }
    const float rstd = 1.0f / sqrtf(block_sum(q, red) / (float)p.d + p.eps);
#pragma unroll
    for (int o = 0; o < 2; o++) {
        if (!p.w[o]) continue;
        const T *w = static_cast<const T *>(p.w[o]);
        T *out = static_cast<T *>(p.out[o]) + (size_t)blockIdx.x * p.ldo;
        for (int i = tid; i < p.d; i += blockDim.x) out[i] = from_f32<T>((row[i] - mean) * rstd * to_f32(w[i]));
    }
}

// Embedding rows into every residual stream, and the first sublayer's input.
template <typename T>
__global__ void embed_streams_kernel(const T *__restrict__ table, int64_t pitch, int vocab, int d, const int *__restrict__ ids,
                                     const __grid_constant__ StreamsOut st) {
    constexpr int N = Vec<T>::N;
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * N, r = blockIdx.y;
    float w[N], b[N];
    if (i < d) {  // weights: rows are padded to whole pieces
        unpack(__ldg(reinterpret_cast<const uint4 *>(static_cast<const T *>(st.w) + i)), w);
        unpack(__ldg(reinterpret_cast<const uint4 *>(static_cast<const T *>(st.b) + i)), b);
    }
    pdl_enter();  // ids are written by the previous step's sampling kernel
    if (i >= d) return;
    int id = ids[r];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);  // ids are validated on the host; never read outside
    float f[N], sum = 0.f;
    unpack(__ldg(reinterpret_cast<const uint4 *>(table + (size_t)id * pitch + i)), f);
    for (int s = 0; s < st.n; s++) sum += st.in[s];
    float *x = st.x + (size_t)r * d + i;
    T *h = static_cast<T *>(st.h) + (size_t)r * st.ldh + i;
    if ((d & 3) == 0 && i + N <= d) {
        for (int s = 0; s < st.n; s++)
#pragma unroll
            for (int e = 0; e < N; e += 4)
                *reinterpret_cast<float4 *>(x + s * st.plane + e) = make_float4(f[e], f[e + 1], f[e + 2], f[e + 3]);
#pragma unroll
        for (int e = 0; e < N; e += 4) {
            float v[4];
#pragma unroll
            for (int j = 0; j < 4; j++) v[j] = tanh_norm(sum * f[e + j], st.alpha, w[e + j], b[e + j]);
            store4(h + e, v);
        }
    } else {
#pragma unroll
        for (int e = 0; e < N; e++)
            if (i + e < d) {
                for (int s = 0; s < st.n; s++) x[s * st.plane + e] = f[e];
                h[e] = from_f32<T>(tanh_norm(sum * f[e], st.alpha, w[e], b[e]));
            }
    }
}

template <typename T>
__global__ void streams_norm_kernel(const __grid_constant__ StreamsOut st, int d, const int *__restrict__ rows) {
    pdl_enter();
    const int i = blockIdx.x * blockDim.x + threadIdx.x, src = rows ? rows[blockIdx.y] : blockIdx.y;
    if (i >= d) return;
    float u = 0.f;
    for (int s = 0; s < st.n; s++) u = fmaf(st.in[s], __ldcg(st.x + s * st.plane + (size_t)src * d + i), u);
    static_cast<T *>(st.h)[(size_t)blockIdx.y * st.ldh + i] =
        from_f32<T>(tanh_norm(u, st.alpha, to_f32(static_cast<const T *>(st.w)[i]), to_f32(static_cast<const T *>(st.b)[i])));
}

// One CTA per row: RMS norm of all query heads at once and of all key heads at once, rotation of
// the first `rot` values of every head, queries to q_out, keys and raw keys (= values) to the cache.
template <typename T>
__global__ void __launch_bounds__(256) qk_rotate_kernel(const RotParams p) {
    extern __shared__ float cs[];  // [rot / 2] cos, [rot / 2] sin
    __shared__ float red[33];
    pdl_enter();
    const int tid = threadIdx.x, r = blockIdx.x;
    const T *q = static_cast<const T *>(p.q) + (size_t)r * p.ldq, *k = static_cast<const T *>(p.k) + (size_t)r * p.ldk;
    const int pos = p.pos[r], nq = p.H * p.D, nk = p.G * p.D, half = p.rot / 2;
    float *sn = cs + half;
    for (int i = tid; i < half; i += blockDim.x) sincosf((float)pos * p.freq[i], &sn[i], &cs[i]);
    float s = 0.f;
    for (int i = tid; i < nq; i += blockDim.x) {
        const float v = to_f32(q[i]);
        s += v * v;
    }
    const float rq = 1.0f / sqrtf(block_sum(s, red) / (float)nq + p.eps);
    s = 0.f;
    for (int i = tid; i < nk; i += blockDim.x) {
        const float v = to_f32(k[i]);
        s += v * v;
    }
    const float rk = 1.0f / sqrtf(block_sum(s, red) / (float)nk + p.eps);  // also a barrier behind cs / sn
    auto value = [&](const T *src, const void *w, float scale, int head, int e) {
        auto norm = [&](int at) { return to_f32(src[at]) * scale * to_f32(static_cast<const T *>(w)[at]); };
        const int at = head * p.D + e;
        if (e >= p.rot) return norm(at);
        const float v = norm(at);
        return e < half ? v * cs[e] - norm(at + half) * sn[e] : v * cs[e - half] + norm(at - half) * sn[e - half];
    };
    T *qo = static_cast<T *>(p.q_out) + (size_t)r * p.H * p.Dp;
    for (int i = tid; i < p.H * p.Dp; i += blockDim.x) {
        const int head = i / p.Dp, e = i - head * p.Dp;
        qo[i] = from_f32<T>(e < p.D ? value(q, p.qn, rq, head, e) : 0.f);
    }
    if (pos < 0 || pos >= p.max_seq) {  // a cache row that does not exist: nothing is written, the host hears about it
        if (tid == 0 && atomicCAS(&p.status->code, 0, TLC_DEV_INDEX) == 0) p.status->where = 401;
        return;
    }
    const size_t base = ((size_t)p.slot[r] * p.max_seq + pos) * p.G * p.Dp;
    T *kc = static_cast<T *>(p.kc) + base, *vc = static_cast<T *>(p.vc) + base;
    for (int i = tid; i < p.G * p.Dp; i += blockDim.x) {
        const int head = i / p.Dp, e = i - head * p.Dp;
        kc[i] = from_f32<T>(e < p.D ? value(k, p.kn, rk, head, e) : 0.f);
        vc[i] = e < p.D ? k[head * p.D + e] : from_f32<T>(0.f);
    }
}

// The same with 16-byte pieces, for bf16 heads of whole pieces whose rotated halves are whole pieces.
// A unit is two pieces that turn against each other, or one piece behind the rotated part.
__global__ void __launch_bounds__(256) qk_rotate_pieces_kernel(const RotParams p) {
    extern __shared__ float cs[];  // [rot / 2] cos, [rot / 2] sin
    __shared__ float red[33];
    pdl_enter();
    const int tid = threadIdx.x, r = blockIdx.x;
    const bf16 *q = static_cast<const bf16 *>(p.q) + (size_t)r * p.ldq, *k = static_cast<const bf16 *>(p.k) + (size_t)r * p.ldk;
    const int pos = p.pos[r], nq = p.H * p.D, nk = p.G * p.D, half = p.rot / 2;
    float *sn = cs + half;
    for (int i = tid; i < half; i += blockDim.x) sincosf((float)pos * p.freq[i], &sn[i], &cs[i]);
    auto squares = [&](const bf16 *x, int n) {
        float s = 0.f;
        for (int i = tid; i < n / 8; i += blockDim.x) {
            float f[8];
            unpack(*(reinterpret_cast<const uint4 *>(x) + i), f);
#pragma unroll
            for (int e = 0; e < 8; e++) s += f[e] * f[e];
        }
        return s;
    };
    const float sq = squares(q, nq), sk = squares(k, nk);
    const float rq = 1.0f / sqrtf(block_sum(sq, red) / (float)nq + p.eps);
    const float rk = 1.0f / sqrtf(block_sum(sk, red) / (float)nk + p.eps);  // also a barrier behind cs / sn
    const bool in_cache = pos >= 0 && pos < p.max_seq;
    if (!in_cache && tid == 0 && atomicCAS(&p.status->code, 0, TLC_DEV_INDEX) == 0) p.status->where = 401;
    const size_t base = ((size_t)p.slot[r] * p.max_seq + (in_cache ? pos : 0)) * p.G * p.D;
    bf16 *kc = static_cast<bf16 *>(p.kc) + base, *vc = static_cast<bf16 *>(p.vc) + base;
    bf16 *qo = static_cast<bf16 *>(p.q_out) + (size_t)r * nq;
    const int turning = half / 8, units = turning + (p.D - p.rot) / 8;  // per head
    const int all = (in_cache ? p.H + p.G : p.H) * units;
    for (int u = tid; u < all; u += blockDim.x) {
        const int head = u / units, i = u - head * units;
        const bool is_q = head < p.H;
        const int hb = (is_q ? head : head - p.H) * p.D, e = i < turning ? 8 * i : p.rot + 8 * (i - turning);
        const bf16 *src = (is_q ? q : k) + hb, *w = static_cast<const bf16 *>(is_q ? p.qn : p.kn) + hb;
        const float scale = is_q ? rq : rk;
        bf16 *dst = (is_q ? qo : kc) + hb;
        const uint4 raw0 = *reinterpret_cast<const uint4 *>(src + e);
        float a[8], wa[8];
        unpack(raw0, a);
        unpack(__ldg(reinterpret_cast<const uint4 *>(w + e)), wa);
#pragma unroll
        for (int j = 0; j < 8; j++) a[j] = a[j] * scale * wa[j];
        if (!is_q) *reinterpret_cast<uint4 *>(vc + hb + e) = raw0;
        if (i < turning) {
            const uint4 raw1 = *reinterpret_cast<const uint4 *>(src + e + half);
            float b[8], wb[8];
            unpack(raw1, b);
            unpack(__ldg(reinterpret_cast<const uint4 *>(w + e + half)), wb);
            if (!is_q) *reinterpret_cast<uint4 *>(vc + hb + e + half) = raw1;
#pragma unroll
            for (int j = 0; j < 8; j++) {
                const float x = a[j], y = b[j] * scale * wb[j];
                a[j] = x * cs[e + j] - y * sn[e + j];
                b[j] = y * cs[e + j] + x * sn[e + j];
            }
            store4(dst + e + half, *reinterpret_cast<const float(*)[4]>(b));
            store4(dst + e + half + 4, *reinterpret_cast<const float(*)[4]>(b + 4));
        }
        store4(dst + e, *reinterpret_cast<const float(*)[4]>(a));
        store4(dst + e + 4, *reinterpret_cast<const float(*)[4]>(a + 4));
    }
}

// One warp per token: the `top` largest sigmoid scores, the lowest index of equals first.
__global__ void route_kernel(const RouteParams p) {
    extern __shared__ float all[];
    pdl_enter();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = blockIdx.x * (blockDim.x >> 5) + warp;
    if (r >= p.m) return;
    float *score = all + (size_t)warp * p.experts;
    for (int e = lane; e < p.experts; e += 32) score[e] = sigmoid_f(p.logits[(size_t)r * p.ld + e]);
    __syncwarp();
    for (int t = 0; t < p.top; t++) {
        float best = -1.f;
        int bi = p.experts;
        for (int e = lane; e < p.experts; e += 32)
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
        if (bi >= p.experts) bi = 0;  // scores that are not numbers: stay inside the tables
        if (lane == 0) {
            score[bi] = -2.f;
            p.chosen[(size_t)r * p.top + t] = bi;
            p.weight[(size_t)r * p.top + t] = best;
            p.rank[(size_t)r * p.top + t] = atomicAdd(p.count + bi, 1);
        }
        __syncwarp();
    }
}

// Rows in the order of their experts: CTA r copies row r to its `top` places.
template <typename T>
__global__ void __launch_bounds__(256) permute_kernel(const PermuteParams p) {
    extern __shared__ int start[];  // [experts + 1]
    pdl_enter();
    const int tid = threadIdx.x, r = blockIdx.x;
    if (tid < 32) {  // exclusive sums of the experts' row counts, 32 at a time
        int carry = 0;
        for (int e0 = 0; e0 < p.experts; e0 += 32) {
            const int e = e0 + tid;
            const int c = e < p.experts ? p.count[e] : 0;
            int incl = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int t = __shfl_up_sync(0xffffffffu, incl, o);
                if (tid >= o) incl += t;
            }
            if (e < p.experts) start[e] = carry + incl - c;
            carry += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (tid == 0) start[p.experts] = carry;
    }
    __syncthreads();
    if (r == 0)
        for (int e = tid; e <= p.experts; e += blockDim.x) p.off[e] = start[e];
    for (int t = 0; t < p.top; t++) {
        const int at = r * p.top + t;
        const int dst = start[p.chosen[at]] + p.rank[at];
        if (tid == 0) {
            p.place[at] = dst;
            p.scale[dst] = p.weight[at];
        }
        // rows are whole 16-byte pieces (ldh is padded)
        const uint4 *src = reinterpret_cast<const uint4 *>(static_cast<const T *>(p.h) + (size_t)r * p.ldh);
        uint4 *to = reinterpret_cast<uint4 *>(static_cast<T *>(p.hp) + (size_t)dst * p.ldh);
        for (int i = tid; i < p.ldh / Vec<T>::N; i += blockDim.x) to[i] = src[i];
    }
}

}  // namespace

#define TLC_LAUNCHED(ctx, le, what)                                                            \
    do {                                                                                       \
        if ((le) != cudaSuccess) {                                                             \
            cudaGetLastError();                                                                \
            return tlc_fail(TLC_ERR_CUDA, what " launch failed: %s", cudaGetErrorString(le));  \
        }                                                                                      \
        TLC_CHECK_LAUNCH(ctx);                                                                 \
    } while (0)

template <typename T>
int32_t launch_embed(tlc_ctx *ctx, const tlc_qtensor *table, const int *ids, int m, float *x) {
    const int d = (int)table->n_cols, per = (d + 256 * Vec<T>::N - 1) / (256 * Vec<T>::N);
    cudaError_t le = tlc_launch_pdl(ctx, embed_rows_kernel<T>, dim3(per, m), dim3(256), 0, static_cast<const T *>(table->data),
                                    (int64_t)(table->row_pitch / sizeof(T)), (int)table->n_rows, d, ids, x);
    TLC_LAUNCHED(ctx, le, "embedding");
    return TLC_OK;
}

template <typename T>
int32_t launch_embed_streams(tlc_ctx *ctx, const tlc_qtensor *table, const int *ids, int m, const StreamsOut &st) {
    const int d = (int)table->n_cols, threads = 128, per = (d + threads * Vec<T>::N - 1) / (threads * Vec<T>::N);
    cudaError_t le = tlc_launch_pdl(ctx, embed_streams_kernel<T>, dim3(per, m), dim3(threads), 0, static_cast<const T *>(table->data),
                                    (int64_t)(table->row_pitch / sizeof(T)), (int)table->n_rows, d, ids, st);
    TLC_LAUNCHED(ctx, le, "embedding");
    return TLC_OK;
}

template <typename T>
int32_t launch_streams_norm(tlc_ctx *ctx, const StreamsOut &st, int width, const int *rows, int m) {
    cudaError_t le = tlc_launch_pdl(ctx, streams_norm_kernel<T>, dim3((width + 255) / 256, m), dim3(256), 0, st, width, rows);
    TLC_LAUNCHED(ctx, le, "streams norm");
    return TLC_OK;
}

template <typename T>
int32_t launch_norm(tlc_ctx *ctx, const NormParams &p) {
    const size_t smem = (size_t)p.d * sizeof(float);
    static bool done[64] = {};
    if (!done[ctx->device & 63]) {
        TLC_CUDA(cudaFuncSetAttribute(norm_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        done[ctx->device & 63] = true;
    }
    TLC_REQUIRE(smem <= 200 * 1024, TLC_ERR_INVALID_OPERATION, "layer norm over %d values does not fit the shared memory", p.d);
    cudaError_t le = tlc_launch_pdl(ctx, norm_rows_kernel<T>, dim3(p.m), dim3(256), smem, p);
    TLC_LAUNCHED(ctx, le, "layer norm");
    return TLC_OK;
}

template <typename T>
int32_t launch_qk_rotate(tlc_ctx *ctx, const RotParams &p, int m) {
    if (sizeof(T) == 2 && p.D % 8 == 0 && p.rot % 16 == 0) {
        cudaError_t le = tlc_launch_pdl(ctx, qk_rotate_pieces_kernel, dim3(m), dim3(256), (size_t)p.rot * sizeof(float) + 16, p);
        TLC_LAUNCHED(ctx, le, "query/key norm");
        return TLC_OK;
    }
    cudaError_t le = tlc_launch_pdl(ctx, qk_rotate_kernel<T>, dim3(m), dim3(256), (size_t)p.rot * sizeof(float) + 16, p);
    TLC_LAUNCHED(ctx, le, "query/key norm");
    return TLC_OK;
}

int32_t launch_route(tlc_ctx *ctx, const RouteParams &p) {
    const int warps = p.experts > 1024 ? 1 : 8;
    cudaError_t le = tlc_launch_pdl(ctx, route_kernel, dim3((p.m + warps - 1) / warps), dim3(32 * warps),
                                    (size_t)warps * p.experts * sizeof(float), p);
    TLC_LAUNCHED(ctx, le, "router");
    return TLC_OK;
}

template <typename T>
int32_t launch_permute(tlc_ctx *ctx, const PermuteParams &p) {
    cudaError_t le = tlc_launch_pdl(ctx, permute_kernel<T>, dim3(p.m), dim3(256), ((size_t)p.experts + 1) * sizeof(int), p);
    TLC_LAUNCHED(ctx, le, "expert permutation");
    return TLC_OK;
}

template int32_t launch_embed<bf16>(tlc_ctx *, const tlc_qtensor *, const int *, int, float *);
template int32_t launch_embed<float>(tlc_ctx *, const tlc_qtensor *, const int *, int, float *);
template int32_t launch_embed_streams<bf16>(tlc_ctx *, const tlc_qtensor *, const int *, int, const StreamsOut &);
template int32_t launch_embed_streams<float>(tlc_ctx *, const tlc_qtensor *, const int *, int, const StreamsOut &);
template int32_t launch_streams_norm<bf16>(tlc_ctx *, const StreamsOut &, int, const int *, int);
template int32_t launch_streams_norm<float>(tlc_ctx *, const StreamsOut &, int, const int *, int);
template int32_t launch_norm<bf16>(tlc_ctx *, const NormParams &);
template int32_t launch_norm<float>(tlc_ctx *, const NormParams &);
template int32_t launch_qk_rotate<bf16>(tlc_ctx *, const RotParams &, int);
template int32_t launch_qk_rotate<float>(tlc_ctx *, const RotParams &, int);
template int32_t launch_permute<bf16>(tlc_ctx *, const PermuteParams &);
template int32_t launch_permute<float>(tlc_ctx *, const PermuteParams &);

}  // namespace tlc_dense
