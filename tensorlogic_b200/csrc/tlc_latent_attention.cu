// Latent attention, absorbed form: the cache holds one latent and one rotated key part per token, and
// all heads read the same rows.
//
//   latent_rows_kernel<T>     many rows: norm of the query latents, norm / rotation / append of the
//                             key latents.
//   latent_query_kernel<T>    per (row, head): query projection (one-row form: a cluster shares the head's
//                             rows of W_uq and exchanges the results through distributed shared memory),
//                             rotation, q' = W_uk^T q.  In the one-row form one more CTA appends the row's
//                             latent to the cache.
//   latent_scan_kernel<NT>    bf16: 16 heads of one row against a stretch of the cache, tensor cores; the
//                             keys' first kp columns are the values too, so a tile is fetched once.
//   latent_scan_fma_kernel<T> the same on the FMA pipes: f32, and latents above 512.
//   latent_value_kernel<T>    merges the stretches, adds the sink, applies W_uv.
//
// Scores, statistics and weights are f32; a weight enters the tensor-core product as the sum of two bf16
// numbers (high and low part).
#include <algorithm>

#include "tlc_dense.cuh"
#include "tlc_mma.cuh"
#include "tlc_stream.cuh"

namespace tlc_dense {

namespace {

constexpr int kQueryThreads = 512, kScanThreads = 512, kValueThreads = 512;
constexpr int kKeys = 64;       // keys per tile
constexpr int kTileHeads = 16;
constexpr int kMaxSplits = 64;
constexpr size_t kScanSmem = 216 * 1024;  // dynamic; the scores and factors of a tile come on top
constexpr int kPPitch = kKeys + 8;
constexpr float kLog2e = 1.44269504088896340736f;

__device__ __forceinline__ uint4 load_nc(const void *p) { return __ldg(static_cast<const uint4 *>(p)); }

// The rotated pair i at `pos`: (u, v) -> (u cos - v sin, v cos + u sin).
__device__ __forceinline__ float2 rotate_pair(float u, float v, int pos, float freq) {
    float sn, cs;
    sincosf((float)pos * freq, &sn, &cs);
    return make_float2(u * cs - v * sn, v * cs + u * sn);
}

// 1 / root mean square of n values of a row padded to whole pieces, by one warp.
template <typename T>
__device__ __forceinline__ float warp_rms(const T *z, int n, float eps, int lane) {
    constexpr int N = Vec<T>::N;
    float s = 0.f;
#pragma unroll 4
    for (int c = lane; N * c < n; c += 32) {
        float f[N];
        unpack(__ldcg(reinterpret_cast<const uint4 *>(z) + c), f);
#pragma unroll
        for (int e = 0; e < N; e++) s += N * c + e < n ? f[e] * f[e] : 0.f;
    }
    return 1.0f / sqrtf(warp_sum(s) / (float)n + eps);
}
// out = z * rstd * w in whole pieces; w is padded with zeros.
template <typename T>
__device__ __forceinline__ void warp_scale(const T *z, const T *w, T *out, int n, float rstd, int lane) {
    constexpr int N = Vec<T>::N;
#pragma unroll 4
    for (int c = lane; N * c < n; c += 32) {
        float f[N], g[N];
        unpack(__ldcg(reinterpret_cast<const uint4 *>(z) + c), f);
        unpack(load_nc(w + N * c), g);
        union { uint4 v; T t[N]; } o;
#pragma unroll
        for (int e = 0; e < N; e++) o.t[e] = from_f32<T>(N * c + e < n ? f[e] * rstd * g[e] : 0.f);
        reinterpret_cast<uint4 *>(out)[c] = o.v;
    }
}

// Row r's latent, normalized, and its rotated key part into the cache.  One warp.
template <typename T>
__device__ void append_latent(const LatentParams &p, int r, int lane) {
    const T *z = static_cast<const T *>(p.ckv_raw) + (size_t)r * p.ldckv;
    const int pos = p.pos[r];
    if (pos < 0 || pos >= p.max_seq) {  // a cache row that does not exist: nothing is written, the host hears about it
        if (lane == 0 && atomicCAS(&p.status->code, 0, TLC_DEV_INDEX) == 0) p.status->where = 411;
        return;
    }
    T *row = static_cast<T *>(p.cache) + ((size_t)p.slot[r] * p.max_seq + pos) * p.row;
    warp_scale(z, static_cast<const T *>(p.dkv_norm), row, p.KR, warp_rms(z, p.KR, p.eps, lane), lane);
    for (int i = lane; i < (p.row - p.kp) / 2; i += 32) {
        float2 v = make_float2(0.f, 0.f);
        if (2 * i < p.R) v = rotate_pair(to_f32(z[p.KR + 2 * i]), to_f32(z[p.KR + 2 * i + 1]), pos, p.freq[i]);
        row[p.kp + 2 * i] = from_f32<T>(v.x);
        row[p.kp + 2 * i + 1] = from_f32<T>(v.y);
    }
}

// A warp per (row, latent of the queries or of the keys).
template <typename T>
__global__ void __launch_bounds__(256) latent_rows_kernel(const __grid_constant__ LatentParams p) {
    pdl_enter();
    const int w = blockIdx.x * 8 + (threadIdx.x >> 5), r = w >> 1, lane = threadIdx.x & 31;
    if (r >= p.m) return;
    if (w & 1) {
        append_latent<T>(p, r, lane);
    } else {
        const T *z = static_cast<const T *>(p.cq_raw) + (size_t)r * p.ldcq;
        warp_scale(z, static_cast<const T *>(p.dq_norm), static_cast<T *>(p.cq) + (size_t)r * p.ldcq, p.QR, warp_rms(z, p.QR, p.eps, lane), lane);
    }
}

__device__ __forceinline__ void store_remote_f32(float *at, int rank, float v) {
    uint32_t dst;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dst) : "r"((uint32_t)__cvta_generic_to_shared(at)), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(v) : "memory");
}

// Grid (C, H [+ 1: the append], rows); the C CTAs of a head are a cluster when p.q is null.
template <typename T>
__global__ void __launch_bounds__(kQueryThreads, 2) latent_query_kernel(const __grid_constant__ LatentParams p, int split) {
    constexpr int N = Vec<T>::N, KEPT = 4;
    extern __shared__ __align__(16) float smem[];
    __shared__ float red[33];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, C = gridDim.x, rank = blockIdx.x, head = blockIdx.y,
              r = blockIdx.z;
    if (head == p.H) {
        pdl_enter();
        if (rank == 0 && warp == 0) append_latent<T>(p, r, lane);
        return;
    }
    const int DR = p.D + p.R, qpieces = (p.QR + N - 1) / N, rows = (DR + C - 1) / C;
    float *qs = smem;                               // [DR]: the head's query
    float *cq = qs + ((DR + 3) & ~3);               // [qpieces * N], in the places of put_piece
    float *sums = cq + (p.q ? 0 : qpieces * N);     // [kQueryThreads][N], before that [rows][split]
    const bool cluster = !p.q && C > 1;
    if (cluster) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");  // this CTA is running
    // latent columns of this CTA, in pieces; a thread holds one piece of columns and every `groups`-th d
    const T *uk = static_cast<const T *>(p.uk) + (size_t)head * p.D * p.uk_pitch;
    const int pieces = (p.KR + N - 1) / N, per = (pieces + C - 1) / C;
    const int p_lo = rank * per < pieces ? rank * per : pieces, p_hi = p_lo + per < pieces ? p_lo + per : pieces;
    const int np = p_hi - p_lo < kQueryThreads ? p_hi - p_lo : kQueryThreads, groups = np > 0 ? kQueryThreads / np : 0;
    const int g = np > 0 ? tid / np : 0, c_own = p_lo + tid - g * np;
    const int pos = p.pos[r];  // written at least two kernels ago
    const int lo = rank * rows, hi = lo + rows < DR ? lo + rows : DR;
    const T *uq = static_cast<const T *>(p.uq) + (size_t)head * DR * p.uq_pitch;
    // weights are never written: they can be on their way before the input exists
    if (!p.q)
        for (int i = lo + tid; i < hi; i += kQueryThreads) prefetch_l2(uq + (size_t)i * p.uq_pitch, (uint32_t)(qpieces * 16));
    if (p_hi > p_lo)
        for (int i = tid; i < p.D; i += kQueryThreads) prefetch_l2(uk + (size_t)i * p.uk_pitch + p_lo * N, (uint32_t)((p_hi - p_lo) * 16));
    float sn = 0.f, cs = 1.f;  // of pair `tid` (more pairs than threads: made where they are used)
    if (rank == 0 && 2 * tid < p.R) sincosf((float)pos * p.freq[tid], &sn, &cs);
    uint4 kept[KEPT];
    auto keep = [&] {  // the first rows of W_uk, on their way while the CTAs exchange the query
#pragma unroll
        for (int i = 0; i < KEPT; i++)
            kept[i] = g < groups && g + i * groups < p.D
                          ? load_weight(reinterpret_cast<const uint4 *>(uk + (size_t)(g + i * groups) * p.uk_pitch) + c_own)
                          : make_uint4(0u, 0u, 0u, 0u);
    };
    pdl_enter();
    if (p.q) {
        keep();
        const T *q = static_cast<const T *>(p.q) + (size_t)r * p.ldq + (size_t)head * DR;
        for (int i = tid; i < DR; i += kQueryThreads) qs[i] = to_f32(q[i]);
        __syncthreads();
    } else {
        const T *z = static_cast<const T *>(p.cq_raw) + (size_t)r * p.ldcq;
        float s = 0.f;
        for (int c = tid; c < qpieces; c += kQueryThreads) {  // rows are padded to whole pieces, with anything
            float f[N];
            unpack(__ldcg(reinterpret_cast<const uint4 *>(z) + c), f);
#pragma unroll
            for (int e = 0; e < N; e++) {
                if (N * c + e >= p.QR) f[e] = 0.f;
                s += f[e] * f[e];
            }
            put_piece<T>(cq, c, qpieces, f);
        }
        const float rstd = 1.0f / sqrtf(block_sum(s, red) / (float)p.QR + p.eps);
        for (int c = tid; c < qpieces; c += kQueryThreads) {  // the thread's own pieces
            float f[N], w[N];
            get_piece<T>(cq, c, qpieces, f);
            unpack(load_nc(static_cast<const T *>(p.dq_norm) + c * N), w);
#pragma unroll
            for (int e = 0; e < N; e++) f[e] *= rstd * w[e];
            put_piece<T>(cq, c, qpieces, f);
        }
        __syncthreads();
        const int share = (qpieces + split - 1) / split;
        if (hi > lo)
            stream_items<T, kQueryThreads / 32>(hi - lo, split, cq, cq + 4 * qpieces, sums, [&](int i, int t) {
                Item it;
                it.w = reinterpret_cast<const uint4 *>(uq + (size_t)(lo + i) * p.uq_pitch);
                share_of(share, qpieces, t, it);
                it.shift = 0;
                it.slot = i * split + t;
                it.scale = 1.f;
                return it;
            });
        keep();
        __syncthreads();
        if (cluster) asm volatile("barrier.cluster.wait.aligned;" ::: "memory");  // every peer is running
        for (int i = tid; i < (hi - lo) * C; i += kQueryThreads) {
            const int row = i / C, peer = i - row * C;
            float a = 0.f;
            for (int t = 0; t < split; t++) a += sums[row * split + t];
            if (cluster)
                store_remote_f32(qs + lo + row, peer, a);
            else
                qs[lo + row] = a;
        }
        if (cluster) {
            asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
            asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
        } else {
            __syncthreads();
        }
    }
    T *out = static_cast<T *>(p.ql) + ((size_t)r * p.H + head) * p.row;
    if (rank == 0) {
        for (int i = pieces * N + tid; i < p.kp; i += kQueryThreads) out[i] = from_f32<T>(0.f);
        for (int i = tid; i < (p.row - p.kp) / 2; i += kQueryThreads) {
            float2 v = make_float2(0.f, 0.f);
            if (2 * i < p.R) {
                const float u = qs[p.D + 2 * i], w = qs[p.D + 2 * i + 1];
                v = i == tid ? make_float2(u * cs - w * sn, w * cs + u * sn) : rotate_pair(u, w, pos, p.freq[i]);
            }
            out[p.kp + 2 * i] = from_f32<T>(v.x);
            out[p.kp + 2 * i + 1] = from_f32<T>(v.y);
        }
    }
    // q'[column] = sum_d q[d] W_uk[d][column]
    for (int c0 = p_lo; c0 < p_hi; c0 += np) {
        const int c = c_own + c0 - p_lo, width = p_hi - c0 < np ? p_hi - c0 : np;  // pieces of this turn
        float acc[N];
#pragma unroll
        for (int e = 0; e < N; e++) acc[e] = 0.f;
        auto add = [&](const uint4 &v, int d) {
            float f[N];
            unpack(v, f);  // rows are padded with zeros
            const float x = qs[d];
#pragma unroll
            for (int e = 0; e < N; e++) acc[e] = fmaf(f[e], x, acc[e]);
        };
        if (g < groups && c < p_hi) {
            int d = g;
            if (c0 == p_lo)
#pragma unroll
                for (int i = 0; i < KEPT; i++, d += groups)
                    if (d < p.D) add(kept[i], d);
#pragma unroll 4
            for (; d < p.D; d += groups) add(load_weight(reinterpret_cast<const uint4 *>(uk + (size_t)d * p.uk_pitch) + c), d);
        }
#pragma unroll
        for (int e = 0; e < N; e += 4)
            *reinterpret_cast<float4 *>(sums + tid * N + e) = make_float4(acc[e], acc[e + 1], acc[e + 2], acc[e + 3]);
        __syncthreads();
        // `parts` threads per column, each every parts-th group, then one
        const int columns = width * N, parts = columns < kQueryThreads ? kQueryThreads / columns : 1;
        if (parts > 1) {
            const int part = tid / columns, i = tid - part * columns;
            float a = 0.f;
            if (part < parts)
                for (int j = part; j < groups; j += parts) a += sums[(size_t)j * np * N + i];
            __syncthreads();
            sums[tid] = a;
            __syncthreads();
            if (tid < columns) {
                for (int j = 1; j < parts; j++) a += sums[j * columns + tid];
                out[c0 * N + tid] = from_f32<T>(a);
            }
        } else {
            for (int i = tid; i < columns; i += kQueryThreads) {
                float a = 0.f;
                for (int j = 0; j < groups; j++) a += sums[(size_t)j * np * N + i];
                out[c0 * N + i] = from_f32<T>(a);
            }
        }
        __syncthreads();
    }
}

// Tiles of the cache the split takes: [lo, hi).
struct Stretch {
    int lo, hi;
    __device__ __forceinline__ Stretch(int keys, int tile, int split, int nsplit) {
        const int tiles = (keys + tile - 1) / tile, per = (tiles + nsplit - 1) / nsplit;
        lo = split * per < tiles ? split * per : tiles;
        hi = lo + per < tiles ? lo + per : tiles;
    }
};

__device__ __forceinline__ int checked_position(const LatentParams &p, int r, int where) {
    int pos = p.pos[r];
    if (pos < 0 || pos >= p.max_seq) {  // outside the cache: cut, and the host hears about it
        if (threadIdx.x == 0 && atomicCAS(&p.status->code, 0, TLC_DEV_INDEX) == 0) p.status->where = where;
        pos = pos < 0 ? 0 : p.max_seq - 1;
    }
    return pos;
}

__host__ __device__ constexpr int scan_pitch(int row) { return ((row + 31) & ~31) + 8; }
__host__ __device__ constexpr size_t scan_smem(int row, int stages) {
    return (size_t)(stages * kKeys + kTileHeads) * scan_pitch(row) * 2 + (size_t)2 * kTileHeads * kPPitch * 2;
}

// Grid (nsplit, 16-head tiles, rows).  Sixteen warps.  Scores: warp w takes eight keys (w mod 8) and half of the
// columns; softmax: warp w takes head w; weighted sum: warp w takes 8 NT columns.
template <int NT>
__global__ void __launch_bounds__(kScanThreads) latent_scan_kernel(const __grid_constant__ LatentParams p) {
    extern __shared__ __align__(128) uint8_t smem_raw[];
    const int pitch = scan_pitch(p.row), tile_elems = kKeys * pitch, chunks = (pitch - 8) / 8, real = p.row / 8;
    bf16 *ks = reinterpret_cast<bf16 *>(smem_raw);  // [2][64][pitch]
    bf16 *qs = ks + 2 * tile_elems;                 // [16][pitch]
    bf16 *ph = qs + kTileHeads * pitch, *pl = ph + kTileHeads * kPPitch;
    __shared__ float sc[2][kTileHeads][kKeys + 2], corr[kTileHeads];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3, mi = lane >> 3;
    const int split = blockIdx.x, head0 = blockIdx.y * kTileHeads, r = blockIdx.z;
    const int heads = p.H - head0 < kTileHeads ? p.H - head0 : kTileHeads;
    const int pos = checked_position(p, r, 412), keys = pos + 1;
    const Stretch st(keys, kKeys, split, p.nsplit);
    const bf16 *cache = static_cast<const bf16 *>(p.cache) + (size_t)p.slot[r] * p.max_seq * p.row;
    auto load_tile = [&](int tile, int stage, int from, int to) {  // keys [from, to) of the tile
        for (int c = tid; c < (to - from) * chunks; c += kScanThreads) {
            const int key = from + c / chunks, part = c % chunks, j = tile * kKeys + key;
            const bool ok = j < keys && part < real;
            cp_async16(ks + stage * tile_elems + key * pitch + part * 8, cache + (ok ? (size_t)j * p.row + part * 8 : 0), ok);
        }
    };
    // Rows of earlier steps do not depend on the kernels in flight; in the one-row form this step's own
    // row is the previous kernel's.
    int early = 0;
    if (st.lo < st.hi) {
        const int settled = (p.q ? keys : pos) - st.lo * kKeys;
        early = settled < 0 ? 0 : settled < kKeys ? settled : kKeys;
        load_tile(st.lo, 0, 0, early);
    }
    pdl_enter();
    for (int c = tid; c < kTileHeads * chunks; c += kScanThreads) {
        const int h = c / chunks, part = c % chunks;
        const bool ok = h < heads && part < real;
        cp_async16(qs + h * pitch + part * 8,
                   static_cast<const bf16 *>(p.ql) + (ok ? ((size_t)r * p.H + head0 + h) * p.row + part * 8 : 0), ok);
    }
    if (st.lo < st.hi) load_tile(st.lo, 0, early, kKeys);
    cp_async_commit();
    float m_run = -INFINITY, l_run = 0.f;  // of head `warp`
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const float scale2 = p.scale * kLog2e;
    const int kpairs = (pitch - 8) / 32, half = warp >> 3, k_lo = half ? (kpairs + 1) / 2 : 0, k_hi = half ? kpairs : (kpairs + 1) / 2;
    const int col0 = warp * 8 * NT;
    for (int tile = st.lo; tile < st.hi; tile++) {
        const int stage = (tile - st.lo) & 1;
        if (tile + 1 < st.hi) {
            load_tile(tile + 1, stage ^ 1, 0, kKeys);
            cp_async_commit();
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const bf16 *kt = ks + stage * tile_elems;
        float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
        const bf16 *qa_at = qs + ((mi & 1) * 8 + (lane & 7)) * pitch + (mi >> 1) * 8;
        const bf16 *kb_at = kt + (8 * (warp & 7) + (lane & 7)) * pitch + mi * 8;
#pragma unroll 3
        for (int kk = k_lo; kk < k_hi; kk++) {
            uint32_t a0[4], a1[4], b[4];
            ldsm_x4(a0, qa_at + 32 * kk);
            ldsm_x4(a1, qa_at + 32 * kk + 16);
            ldsm_x4(b, kb_at + 32 * kk);
            mma_bf16(s, a0, b[0], b[1]);
            mma_bf16(s2, a1, b[2], b[3]);
        }
#pragma unroll
        for (int h = 0; h < 2; h++)
            *reinterpret_cast<float2 *>(&sc[half][g + 8 * h][8 * (warp & 7) + 2 * t]) = make_float2(s[2 * h] + s2[2 * h], s[2 * h + 1] + s2[2 * h + 1]);
        __syncthreads();
        {
            const float2 u = *reinterpret_cast<const float2 *>(&sc[0][warp][2 * lane]), v = *reinterpret_cast<const float2 *>(&sc[1][warp][2 * lane]);
            const int j = tile * kKeys + 2 * lane;
            const float x = j < keys ? (u.x + v.x) * scale2 : -INFINITY, y = j + 1 < keys ? (u.y + v.y) * scale2 : -INFINITY;
            float m = fmaxf(x, y);
#pragma unroll
            for (int o2 = 16; o2 > 0; o2 >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o2));
            m = fmaxf(m, m_run);  // a tile has at least one key: m is finite
            const float c = exp2f(m_run - m), a = exp2f(x - m), b = exp2f(y - m);
            m_run = m;
            l_run = l_run * c + a + b;
            uint32_t hi, lo;
            split_pair(a, b, hi, lo);
            *reinterpret_cast<uint32_t *>(ph + warp * kPPitch + 2 * lane) = hi;
            *reinterpret_cast<uint32_t *>(pl + warp * kPPitch + 2 * lane) = lo;
            if (lane == 0) corr[warp] = c;
        }
        __syncthreads();
        const float c0 = corr[g], c1 = corr[g + 8];
#pragma unroll
        for (int d = 0; d < NT; d++) {
            o[d][0] *= c0;
            o[d][1] *= c0;
            o[d][2] *= c1;
            o[d][3] *= c1;
        }
#pragma unroll
        for (int kk = 0; kk < kKeys / 16; kk++) {
            uint32_t hi[4], lo[4];
            const int at = ((mi & 1) * 8 + (lane & 7)) * kPPitch + 16 * kk + (mi >> 1) * 8;
            ldsm_x4(hi, ph + at);
            ldsm_x4(lo, pl + at);
#pragma unroll
            for (int jd = 0; jd < NT / 2; jd++) {
                if (col0 + 16 * jd >= p.kp) break;
                uint32_t b[4];
                ldsm_x4_trans(b, kt + (16 * kk + (mi & 1) * 8 + (lane & 7)) * pitch + col0 + 16 * jd + (mi >> 1) * 8);
                mma_bf16(o[2 * jd], hi, b[0], b[1]);
                mma_bf16(o[2 * jd + 1], hi, b[2], b[3]);
                mma_bf16(o[2 * jd], lo, b[0], b[1]);
                mma_bf16(o[2 * jd + 1], lo, b[2], b[3]);
            }
        }
        __syncthreads();
    }
    cp_async_wait<0>();
    l_run = warp_sum(l_run);
    if (lane == 0 && warp < heads)
        reinterpret_cast<float2 *>(p.stat)[((size_t)r * p.H + head0 + warp) * p.nsplit + split] = make_float2(m_run, l_run);
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int row = g + 8 * h;
        if (row >= heads) continue;
        float *out = p.part + (((size_t)r * p.nsplit + split) * p.H + head0 + row) * p.kp;
#pragma unroll
        for (int d = 0; d < NT; d++) {
            const int c = col0 + 8 * d + 2 * t;
            if (c < p.kp) *reinterpret_cast<float2 *>(out + c) = make_float2(o[d][2 * h], o[d][2 * h + 1]);
        }
    }
}

constexpr int kFmaCols = 512;

// One warp per (row, head, stretch): 32 keys at a time, a key per lane for the scores, every 32nd column per
// lane for the weighted sum; blockIdx.y: which 512 columns.
template <typename T>
__global__ void __launch_bounds__(128) latent_scan_fma_kernel(const __grid_constant__ LatentParams p) {
    extern __shared__ __align__(16) float smem[];  // [4][row]
    constexpr int N = Vec<T>::N;
    pdl_enter();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long w = (long long)blockIdx.x * 4 + warp;
    if (w >= (long long)p.m * p.H * p.nsplit) return;
    const int head = (int)(w % p.H), split = (int)(w / p.H % p.nsplit), r = (int)(w / p.H / p.nsplit);
    float *q = smem + (size_t)warp * p.row;
    const T *qg = static_cast<const T *>(p.ql) + ((size_t)r * p.H + head) * p.row;
    for (int e = lane; e < p.row; e += 32) q[e] = to_f32(qg[e]);
    __syncwarp();
    int pos = p.pos[r];
    if (pos < 0 || pos >= p.max_seq) {
        if (lane == 0 && atomicCAS(&p.status->code, 0, TLC_DEV_INDEX) == 0) p.status->where = 413;
        pos = pos < 0 ? 0 : p.max_seq - 1;
    }
    const int keys = pos + 1, c0 = blockIdx.y * kFmaCols, cols = p.kp - c0 < kFmaCols ? p.kp - c0 : kFmaCols;
    const Stretch st(keys, 32, split, p.nsplit);
    const T *cache = static_cast<const T *>(p.cache) + (size_t)p.slot[r] * p.max_seq * p.row;
    const float scale2 = p.scale * kLog2e;
    float acc[kFmaCols / 32];
#pragma unroll
    for (int i = 0; i < kFmaCols / 32; i++) acc[i] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;
    for (int tile = st.lo; tile < st.hi; tile++) {
        const int j0 = 32 * tile, n = keys - j0 < 32 ? keys - j0 : 32;
        float s = -INFINITY;
        if (lane < n) {
            const uint4 *k = reinterpret_cast<const uint4 *>(cache + (size_t)(j0 + lane) * p.row);
            s = 0.f;
            for (int c = 0; c < p.row / N; c++) {
                float f[N];
                unpack(k[c], f);
#pragma unroll
                for (int e = 0; e < N; e++) s = fmaf(f[e], q[c * N + e], s);
            }
            s *= scale2;
        }
        float mx = s;
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        const float m_new = fmaxf(m_run, mx), corr = exp2f(m_run - m_new), pr = exp2f(s - m_new);
        l_run = l_run * corr + warp_sum(pr);
        m_run = m_new;
#pragma unroll
        for (int i = 0; i < kFmaCols / 32; i++) acc[i] *= corr;
        for (int j = 0; j < n; j++) {
            const float pj = __shfl_sync(0xffffffffu, pr, j);
            const T *val = cache + (size_t)(j0 + j) * p.row + c0;
#pragma unroll
            for (int i = 0; i < kFmaCols / 32; i++)
                if (32 * i + lane < cols) acc[i] = fmaf(pj, to_f32(val[32 * i + lane]), acc[i]);
        }
    }
    const size_t at = ((size_t)r * p.nsplit + split) * p.H + head;
#pragma unroll
    for (int i = 0; i < kFmaCols / 32; i++)
        if (32 * i + lane < cols) p.part[at * p.kp + c0 + 32 * i + lane] = acc[i];
    if (lane == 0 && c0 == 0) reinterpret_cast<float2 *>(p.stat)[((size_t)r * p.H + head) * p.nsplit + split] = make_float2(m_run, l_run);
}

// Grid (shares of the head's values, H, rows).
template <typename T>
__global__ void __launch_bounds__(kValueThreads, 2) latent_value_kernel(const __grid_constant__ LatentParams p) {
    constexpr int N = Vec<T>::N, WARPS = kValueThreads / 32, KEPT = 2, PARTS = 4;
    extern __shared__ __align__(16) float smem[];
    float *ol = smem, *f = ol + p.kp, *sums = f + ((p.nsplit + 3) & ~3);  // the head's weighted latent; factors; [kValueThreads][4]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, head = blockIdx.y, r = blockIdx.z;
    const int per = (p.V + gridDim.x - 1) / gridDim.x, lo = blockIdx.x * per, hi = lo + per < p.V ? lo + per : p.V;
    const T *uv = static_cast<const T *>(p.uv) + (size_t)head * p.V * p.uv_pitch;
    const int pieces = (p.KR + N - 1) / N;
    // the first weight rows and pieces of this warp, before the input exists
    uint4 kept[KEPT][KEPT];
#pragma unroll
    for (int k = 0; k < KEPT; k++)
#pragma unroll
        for (int u = 0; u < KEPT; u++) {
            const int i = lo + warp + WARPS * k, c = lane + 32 * u;
            kept[k][u] = i < hi && c < pieces ? load_weight(reinterpret_cast<const uint4 *>(uv + (size_t)i * p.uv_pitch) + c)
                                              : make_uint4(0u, 0u, 0u, 0u);
        }
    const float sink = to_f32(static_cast<const T *>(p.sink)[head]) * kLog2e;
    pdl_enter();
    if (lo >= hi) return;
    const float2 *stat = reinterpret_cast<const float2 *>(p.stat) + ((size_t)r * p.H + head) * p.nsplit;
    const float *part = p.part + ((size_t)r * p.nsplit * p.H + head) * p.kp;
    const size_t step = (size_t)p.H * p.kp;
    // a thread adds four columns of every `groups`-th stretch
    const int quads = p.kp / 4 < kValueThreads ? p.kp / 4 : kValueThreads, groups = kValueThreads / quads, g = tid / quads;
    float4 v[PARTS];
#pragma unroll
    for (int i = 0; i < PARTS; i++)
        if (g < groups && g + i * groups < p.nsplit)
            v[i] = __ldcg(reinterpret_cast<const float4 *>(part + (g + i * groups) * step) + (tid - g * quads));
    if (warp == WARPS - 1) {  // factors: exp2(m_s - m) / (sum_s l_s exp2(m_s - m) + exp2(sink - m)); at most 64 stretches
        float2 a = make_float2(-INFINITY, 0.f), b = a;
        if (lane < p.nsplit) a = __ldcg(stat + lane);
        if (lane + 32 < p.nsplit) b = __ldcg(stat + lane + 32);
        float m = fmaxf(fmaxf(a.x, b.x), sink);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        a.x = exp2f(a.x - m);
        b.x = exp2f(b.x - m);
        const float l = warp_sum(a.x * a.y + b.x * b.y) + exp2f(sink - m);
        if (lane < p.nsplit) f[lane] = a.x / l;
        if (lane + 32 < p.nsplit) f[lane + 32] = b.x / l;
    }
    __syncthreads();
    for (int q0 = 0; q0 < p.kp / 4; q0 += quads) {
        const int q = q0 + tid - g * quads;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        auto add = [&](const float4 &w, int s) {
            const float e = f[s];
            a.x = fmaf(e, w.x, a.x);
            a.y = fmaf(e, w.y, a.y);
            a.z = fmaf(e, w.z, a.z);
            a.w = fmaf(e, w.w, a.w);
        };
        if (g < groups && q < p.kp / 4) {
            int s = g;
            if (q0 == 0)
#pragma unroll
                for (int i = 0; i < PARTS; i++, s += groups)
                    if (s < p.nsplit) add(v[i], s);
#pragma unroll 4
            for (; s < p.nsplit; s += groups) add(__ldcg(reinterpret_cast<const float4 *>(part + s * step) + q), s);
        }
        *reinterpret_cast<float4 *>(sums + 4 * tid) = a;
        __syncthreads();
        for (int i = tid; i < 4 * quads && 4 * q0 + i < p.kp; i += kValueThreads) {
            float t = 0.f;
            for (int j = 0; j < groups; j++) t += sums[j * 4 * quads + i];
            ol[4 * q0 + i] = t;
        }
        __syncthreads();
    }
    T *out = static_cast<T *>(p.out) + (size_t)r * p.ldo + (size_t)head * p.V;
    auto dot = [&](const uint4 &w, int c) {
        float x[N], s = 0.f;
        unpack(w, x);  // rows are padded with zeros
#pragma unroll
        for (int e = 0; e < N; e += 4) {
            const float4 o = *reinterpret_cast<const float4 *>(ol + c * N + e);
            s = fmaf(x[e], o.x, s);
            s = fmaf(x[e + 1], o.y, s);
            s = fmaf(x[e + 2], o.z, s);
            s = fmaf(x[e + 3], o.w, s);
        }
        return s;
    };
    auto finish = [&](float acc, int i) {
        acc = warp_sum(acc);
        if (lane == 0) out[i] = from_f32<T>(acc);
    };
#pragma unroll
    for (int k = 0; k < KEPT; k++) {
        const int i = lo + warp + WARPS * k;
        if (i >= hi) break;
        float acc = 0.f;
#pragma unroll
        for (int u = 0; u < KEPT; u++)
            if (lane + 32 * u < pieces) acc += dot(kept[k][u], lane + 32 * u);
        for (int c = lane + 32 * KEPT; c < pieces; c += 32) acc += dot(load_weight(reinterpret_cast<const uint4 *>(uv + (size_t)i * p.uv_pitch) + c), c);
        finish(acc, i);
    }
    for (int i = lo + warp + WARPS * KEPT; i < hi; i += WARPS) {
        float acc = 0.f;
#pragma unroll 4
        for (int c = lane; c < pieces; c += 32) acc += dot(load_weight(reinterpret_cast<const uint4 *>(uv + (size_t)i * p.uv_pitch) + c), c);
        finish(acc, i);
    }
}

int32_t launched(tlc_ctx *ctx, cudaError_t le) {
    if (le != cudaSuccess) {
        cudaGetLastError();
        return tlc_fail(TLC_ERR_CUDA, "latent attention launch failed: %s", cudaGetErrorString(le));
    }
    TLC_CHECK_LAUNCH(ctx);
    return TLC_OK;
}

bool scan_on_tensor_cores(const LatentParams &p, size_t elem) { return elem == 2 && p.kp <= 512 && scan_smem(p.row, 2) <= kScanSmem; }

template <typename K>
int32_t allow_smem(K kernel, bool (&done)[64], int device, size_t bytes) {
    if (done[device & 63]) return TLC_OK;
    TLC_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
    done[device & 63] = true;
    return TLC_OK;
}

template <int NT>
int32_t scan_t(tlc_ctx *ctx, const LatentParams &p) {
    static bool done[64] = {};
    if (int32_t rc = allow_smem(latent_scan_kernel<NT>, done, ctx->device, kScanSmem)) return rc;
    return launched(ctx, tlc_launch_pdl(ctx, latent_scan_kernel<NT>,
                                        dim3((unsigned)p.nsplit, (unsigned)((p.H + kTileHeads - 1) / kTileHeads), (unsigned)p.m),
                                        dim3(kScanThreads), scan_smem(p.row, 2), p));
}

}  // namespace

int latent_splits(const tlc_ctx *ctx, const LatentParams &p) {
    const int per_row = (p.H + kTileHeads - 1) / kTileHeads, tiles = (p.max_seq + kKeys - 1) / kKeys;
    int n = ctx->sm_count / (per_row * p.m);
    n = n < tiles ? n : tiles;
    return n < 1 ? 1 : n > kMaxSplits ? kMaxSplits : n;
}

template <typename T>
int32_t launch_latent_rows(tlc_ctx *ctx, const LatentParams &p) {
    return launched(ctx, tlc_launch_pdl(ctx, latent_rows_kernel<T>, dim3((unsigned)((2 * p.m + 7) / 8)), dim3(256), 0, p));
}

template <typename T>
int32_t launch_latent_query(tlc_ctx *ctx, const LatentParams &p) {
    constexpr int N = Vec<T>::N;
    const int DR = p.D + p.R, qpieces = (p.QR + N - 1) / N;
    // CTAs per head: up to two per SM, at most eight (a portable cluster), no more than pieces of the latent
    int C = 1;
    while (C < 8 && (long)C * (p.H + 1) * p.m <= ctx->sm_count && 2 * C <= p.kp / N) C *= 2;
    const int split = (qpieces + 32 * kBatch - 1) / (32 * kBatch);  // stretches a row of W_uq is cut into
    const size_t area = std::max((size_t)kQueryThreads * N, p.q ? 0 : (size_t)((DR + C - 1) / C) * split);
    const size_t smem = ((size_t)((DR + 3) & ~3) + (p.q ? 0 : (size_t)qpieces * N) + area) * sizeof(float);
    TLC_REQUIRE(smem <= 200 * 1024, TLC_ERR_INVALID_OPERATION, "latent attention: a query latent of %d and heads of %d + %d do not fit",
                p.QR, p.D, p.R);
    static bool done[64] = {};
    if (int32_t rc = allow_smem(latent_query_kernel<T>, done, ctx->device, 200 * 1024)) return rc;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)C, (unsigned)(p.q ? p.H : p.H + 1), (unsigned)p.m);
    cfg.blockDim = dim3(kQueryThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (ctx->use_pdl && ctx->pdl_small) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (!p.q && C > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = (unsigned)C;
        attr[n].val.clusterDim.y = 1;
        attr[n++].val.clusterDim.z = 1;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    return launched(ctx, cudaLaunchKernelEx(&cfg, latent_query_kernel<T>, p, split));
}

template <typename T>
int32_t launch_latent_absorbed(tlc_ctx *ctx, const LatentParams &p) {
    int32_t rc;
    if (scan_on_tensor_cores(p, sizeof(T))) {
        rc = p.kp <= 256 ? scan_t<2>(ctx, p) : scan_t<4>(ctx, p);
    } else {
        const size_t smem = (size_t)4 * p.row * sizeof(float);
        TLC_REQUIRE(smem <= 200 * 1024, TLC_ERR_INVALID_OPERATION, "latent attention: cache rows of %d values do not fit", p.row);
        static bool done[64] = {};
        if ((rc = allow_smem(latent_scan_fma_kernel<T>, done, ctx->device, 200 * 1024))) return rc;
        const long long warps = (long long)p.m * p.H * p.nsplit;
        rc = launched(ctx, tlc_launch_pdl(ctx, latent_scan_fma_kernel<T>,
                                          dim3((unsigned)((warps + 3) / 4), (unsigned)((p.kp + kFmaCols - 1) / kFmaCols)), dim3(128),
                                          smem, p));
    }
    if (rc) return rc;
    const size_t smem = ((size_t)p.kp + ((p.nsplit + 3) & ~3) + 4 * kValueThreads) * sizeof(float);
    TLC_REQUIRE(smem <= 200 * 1024, TLC_ERR_INVALID_OPERATION, "latent attention: a latent of %d values does not fit", p.KR);
    static bool done[64] = {};
    if ((rc = allow_smem(latent_value_kernel<T>, done, ctx->device, 200 * 1024))) return rc;
    int shares = 1;
    while (shares < 8 && (long)2 * shares * p.H * p.m <= ctx->sm_count && 16 * shares <= p.V) shares *= 2;
    return launched(ctx, tlc_launch_pdl(ctx, latent_value_kernel<T>, dim3((unsigned)shares, (unsigned)p.H, (unsigned)p.m),
                                        dim3(kValueThreads), smem, p));
}

template int32_t launch_latent_rows<bf16>(tlc_ctx *, const LatentParams &);
template int32_t launch_latent_rows<float>(tlc_ctx *, const LatentParams &);
template int32_t launch_latent_query<bf16>(tlc_ctx *, const LatentParams &);
template int32_t launch_latent_query<float>(tlc_ctx *, const LatentParams &);
template int32_t launch_latent_absorbed<bf16>(tlc_ctx *, const LatentParams &);
template int32_t launch_latent_absorbed<float>(tlc_ctx *, const LatentParams &);

}  // namespace tlc_dense
