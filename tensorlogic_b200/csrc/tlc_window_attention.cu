// Attention over a sliding window with kept first tokens: the query at position i sees key j <= i
// if i - j < window or j < keep.  Grouped query heads, any head size; scores, softmax statistics
// and weights are f32.
//
//   window_prefill_kernel<D>  bf16, consecutive rows of one sequence: 64 (query, head) rows of one
//                             key/value head per CTA against 64-key tiles; tiles no row of the CTA
//                             can see are never loaded.
//   window_decode_kernel<D>   bf16, one query per sequence: query/key norm and rotation, the cache
//                             append and the attention in one launch.  The visible keys (kept ones,
//                             then the window) are numbered without a gap and shared out over the
//                             CTAs of a cluster; every CTA merges its share of the columns from
//                             what the others pushed into its shared memory.
//   window_rows_kernel<T>     one warp per (row, head), FMA pipes: f32 models and head sizes the
//                             tensor-core forms do not take.
//
// The products run on mma.sync with f32 accumulation.  A weight goes into the P.V product as the
// sum of two bf16 numbers (high and low part), so it keeps 16 bits of mantissa.
#include "tlc_dense.cuh"
#include "tlc_mma.cuh"

namespace tlc_dense {

namespace {

constexpr int kKeys = 64;     // keys per tile
constexpr int kAttn = 128;    // threads

// The visible keys of the query at `pos`, numbered from 0: the kept ones the window does not
// reach, then the window.
struct Visible {
    int kept, first, count;  // first: position of the key numbered `kept`
    __device__ __forceinline__ Visible(int pos, int window, int keep) {
        first = pos - window + 1 > 0 ? pos - window + 1 : 0;
        kept = keep < first ? keep : first;
        count = kept + pos + 1 - first;
    }
    __device__ __forceinline__ int position(int v) const { return v < kept ? v : first + v - kept; }
};

template <int D>
__global__ void __launch_bounds__(kAttn) window_prefill_kernel(const __grid_constant__ WindowAttn p, int slot) {
    constexpr int PITCH = D + 8, TILE = kKeys * PITCH, KSTEPS = D / 16, NDT = D / 8;
    extern __shared__ __align__(128) uint8_t smem_raw[];
    bf16 *ks = reinterpret_cast<bf16 *>(smem_raw);  // [2][TILE]
    bf16 *vs = ks + 2 * TILE;                       // [2][TILE]
    bf16 *qs = vs + 2 * TILE;                       // [64][PITCH]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int hk = blockIdx.y, grp = p.H / p.G;
    const int total = p.m * grp;  // (query, head of the group) rows, heads fastest
    // later rows first: they have the most keys
    const int row0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * 64;
    pdl_enter();
    constexpr int CH = D / 8;
    for (int c = tid; c < 64 * CH; c += kAttn) {
        const int r = c / CH, part = c % CH, fr = row0 + r;
        const int qi = fr / grp, head = hk * grp + fr % grp;
        const bool ok = fr < total && part * 8 < p.Dp;
        cp_async16(qs + r * PITCH + part * 8,
                   static_cast<const bf16 *>(p.q) + (ok ? ((size_t)qi * p.H + head) * p.Dp + part * 8 : 0), ok);
    }
    const bf16 *kbase = static_cast<const bf16 *>(p.kc) + ((size_t)slot * p.max_seq * p.G + hk) * p.Dp;
    const bf16 *vbase = static_cast<const bf16 *>(p.vc) + ((size_t)slot * p.max_seq * p.G + hk) * p.Dp;
    const size_t key_stride = (size_t)p.G * p.Dp;
    const int q_first = p.pos0 + row0 / grp;
    const int last_row = row0 + 63 < total - 1 ? row0 + 63 : total - 1;
    const int q_last = p.pos0 + last_row / grp;
    // tiles: those of the kept keys, then the window's from the first row's edge to the last row
    const int w_tile = (q_first - p.window + 1 > 0 ? q_first - p.window + 1 : 0) / kKeys;
    const int kept_tiles_all = (p.keep + kKeys - 1) / kKeys;
    const int kept_tiles = kept_tiles_all < w_tile ? kept_tiles_all : w_tile;
    const int ntiles = kept_tiles + q_last / kKeys - w_tile + 1;
    auto tile_start = [&](int i) { return (i < kept_tiles ? i : w_tile + i - kept_tiles) * kKeys; };
    auto load_tile = [&](int i, int stage) {
        const int j0 = tile_start(i);
        for (int c = tid; c < kKeys * CH; c += kAttn) {
            const int key = c / CH, part = c % CH;
            const bool ok = j0 + key <= q_last && part * 8 < p.Dp;
            const size_t off = ok ? (size_t)(j0 + key) * key_stride + part * 8 : 0;
            cp_async16(ks + stage * TILE + key * PITCH + part * 8, kbase + off, ok);
            cp_async16(vs + stage * TILE + key * PITCH + part * 8, vbase + off, ok);
        }
        cp_async_commit();
    };
    load_tile(0, 0);
    const int fr[2] = {row0 + 16 * warp + g, row0 + 16 * warp + g + 8};
    const int rpos[2] = {p.pos0 + fr[0] / grp, p.pos0 + fr[1] / grp};
    // positions of this warp's first and last row
    const int wp_first = p.pos0 + (row0 + 16 * warp) / grp, wp_last = p.pos0 + (row0 + 16 * warp + 15) / grp;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    float o[NDT][4];
#pragma unroll
    for (int i = 0; i < NDT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const float scale2 = p.scale * 1.44269504088896340736f;  // exponentials to base 2

    for (int i = 0; i < ntiles; i++) {
        const int stage = i & 1;
        if (i + 1 < ntiles) {
            load_tile(i + 1, stage ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const int j0 = tile_start(i);
        // does any row of this warp see a key of the tile?
        const bool any = j0 <= wp_last && (j0 < p.keep || j0 + kKeys - 1 > wp_first - p.window);
        if (any) {
            const bf16 *kt = ks + stage * TILE, *vt = vs + stage * TILE;
            float s[8][4];
#pragma unroll
            for (int n = 0; n < 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
            const int mi = lane >> 3;
#pragma unroll
            for (int kk = 0; kk < KSTEPS; kk++) {
                uint32_t qa[4];
                ldsm_x4(qa, qs + (16 * warp + (mi & 1) * 8 + (lane & 7)) * PITCH + 16 * kk + (mi >> 1) * 8);
#pragma unroll
                for (int np = 0; np < 4; np++) {
                    uint32_t r[4];
                    ldsm_x4(r, kt + (16 * np + (mi >> 1) * 8 + (lane & 7)) * PITCH + 16 * kk + (mi & 1) * 8);
                    mma_bf16(s[2 * np], qa, r[0], r[1]);
                    mma_bf16(s[2 * np + 1], qa, r[2], r[3]);
                }
            }
            // every row of the warp sees every key: no mask
            const bool all = j0 + kKeys - 1 <= wp_first && (j0 + kKeys <= p.keep || j0 > wp_last - p.window);
            float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int n = 0; n < 8; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    float v = s[n][e] * scale2;
                    if (!all) {
                        const int key = j0 + 8 * n + 2 * t + (e & 1), pos = rpos[e >> 1];
                        if (key > pos || (pos - key >= p.window && key >= p.keep)) v = -INFINITY;
                    }
                    s[n][e] = v;
                    mx[e >> 1] = fmaxf(mx[e >> 1], v);
                }
            float corr[2], base[2];
#pragma unroll
            for (int h = 0; h < 2; h++) {
                mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
                mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
                const float m_new = fmaxf(m_run[h], mx[h]);
                base[h] = m_new == -INFINITY ? 0.f : m_new;
                corr[h] = exp2f(m_run[h] - base[h]);
                m_run[h] = m_new;
            }
            float psum[2] = {0.f, 0.f};
#pragma unroll
            for (int n = 0; n < 8; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    s[n][e] = exp2f(s[n][e] - base[e >> 1]);
                    psum[e >> 1] += s[n][e];
                }
            l_run[0] = l_run[0] * corr[0] + psum[0];
            l_run[1] = l_run[1] * corr[1] + psum[1];
#pragma unroll
            for (int d = 0; d < NDT; d++) {
                o[d][0] *= corr[0];
                o[d][1] *= corr[0];
                o[d][2] *= corr[1];
                o[d][3] *= corr[1];
            }
#pragma unroll
            for (int kp = 0; kp < 4; kp++) {
                uint32_t hi[4], lo[4];
                split_pair(s[2 * kp][0], s[2 * kp][1], hi[0], lo[0]);
                split_pair(s[2 * kp][2], s[2 * kp][3], hi[1], lo[1]);
                split_pair(s[2 * kp + 1][0], s[2 * kp + 1][1], hi[2], lo[2]);
                split_pair(s[2 * kp + 1][2], s[2 * kp + 1][3], hi[3], lo[3]);
#pragma unroll
                for (int jd = 0; jd < KSTEPS; jd++) {
                    uint32_t r[4];
                    ldsm_x4_trans(r, vt + (16 * kp + (mi & 1) * 8 + (lane & 7)) * PITCH + 16 * jd + (mi >> 1) * 8);
                    mma_bf16(o[2 * jd], hi, r[0], r[1]);
                    mma_bf16(o[2 * jd + 1], hi, r[2], r[3]);
                    mma_bf16(o[2 * jd], lo, r[0], r[1]);
                    mma_bf16(o[2 * jd + 1], lo, r[2], r[3]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
        if (fr[h] >= total) continue;
        const float inv = l_run[h] > 0.f ? 1.0f / l_run[h] : 0.f;
        const int qi = fr[h] / grp, head = hk * grp + fr[h] % grp;
        bf16 *out = static_cast<bf16 *>(p.out) + (size_t)qi * p.ldo + (size_t)head * p.D;
        const bool pairs = ((p.D | p.ldo) & 1) == 0;
#pragma unroll
        for (int d = 0; d < NDT; d++) {
            const int e = 8 * d + 2 * t;
            const float a = o[d][2 * h] * inv, b = o[d][2 * h + 1] * inv;
            if (pairs) {
                if (e < p.D) *reinterpret_cast<uint32_t *>(out + e) = pack_bf16(a, b);
            } else {
                if (e < p.D) out[e] = from_f32<bf16>(a);
                if (e + 1 < p.D) out[e + 1] = from_f32<bf16>(b);
            }
        }
    }
}

// Merge area of one CTA: from every split this CTA's columns of the 16 rows, each followed by the
// row's maximum and sum (and two unused floats: rows are whole 16-byte pieces).
__host__ __device__ constexpr int merge_floats(int D, int nsplit) { return nsplit * 16 * (D / nsplit + 4); }
__host__ __device__ constexpr size_t decode_tile_bytes(int D) { return (size_t)4 * kKeys * (D + 8) * 2; }
__host__ __device__ constexpr size_t decode_smem(int D, int nsplit, int half) {
    return decode_tile_bytes(D) + (size_t)16 * (D + 8) * 2 + (size_t)2 * (D + 8) * 2 + (size_t)2 * half * 4 +
           (size_t)merge_floats(D, nsplit) * 4 + 80;
}

__device__ __forceinline__ uint32_t remote_address(uint32_t addr, int rank) {
    uint32_t dst;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dst) : "r"(addr), "r"(rank));
    return dst;
}
__device__ __forceinline__ void store_remote(uint32_t addr, float4 v) {
    asm volatile("st.shared::cluster.v4.f32 [%0], {%1, %2, %3, %4};" ::"r"(addr), "f"(v.x), "f"(v.y), "f"(v.z), "f"(v.w)
                 : "memory");
}
__device__ __forceinline__ void store_remote(uint32_t addr, float2 v) {
    asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(addr), "f"(v.x), "f"(v.y) : "memory");
}
// Two sums over the block at once, the same values in every thread.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2 *red) {
    a = warp_sum(a);
    b = warp_sum(b);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(a, b);
    __syncthreads();
    float2 s = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < kAttn / 32; i++) {
        s.x += red[i].x;
        s.y += red[i].y;
    }
    return s;
}
// Entries a pair unit covers: unit i < rot / 2 turns entries i and i + rot / 2, later units hold two
// neighbours behind the rotated part.
struct Pair {
    int e0, e1;
    bool turn;
    __device__ __forceinline__ Pair(int i, int rot) {
        const int half = rot / 2;
        turn = i < half;
        e0 = turn ? i : rot + 2 * (i - half);
        e1 = turn ? i + half : e0 + 1;
    }
};

template <int D>
__global__ void __launch_bounds__(kAttn) window_decode_kernel(const __grid_constant__ WindowAttn p) {
    constexpr int PITCH = D + 8, TILE = kKeys * PITCH, KSTEPS = D / 16, NDT = D / 8, CH = D / 8;
    extern __shared__ __align__(128) uint8_t smem_raw[];
    bf16 *ks = reinterpret_cast<bf16 *>(smem_raw);
    bf16 *vs = ks + 2 * TILE;
    bf16 *qs = vs + 2 * TILE;           // [16][PITCH]
    bf16 *newk = qs + 16 * PITCH, *newv = newk + PITCH;
    const int half = p.rot / 2;
    float *cs = reinterpret_cast<float *>(newv + PITCH), *sn = cs + half;
    float *merge = reinterpret_cast<float *>((reinterpret_cast<uintptr_t>(sn + half) + 15) & ~(uintptr_t)15);
    __shared__ float2 red[kAttn / 32];
    __shared__ float sm_m[4][16], sm_l[4][16];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int nsplit = p.nsplit;
    const bool cluster = nsplit > 1;
    // tell the peers this CTA is running: its shared memory may be written from now on
    if (cluster) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    const int split = blockIdx.x % nsplit, qt = blockIdx.x / nsplit, hk = blockIdx.y, r = blockIdx.z;
    const int grp = p.H / p.G, heads = grp - 16 * qt < 16 ? grp - 16 * qt : 16;
    // positions were written at least two kernels ago (see the launch-order rule)
    int pos = p.pos[r];
    const int slot = p.slot[r];
    if (pos < 0 || pos >= p.max_seq) {  // outside the cache: cut, and the host hears about it
        if (tid == 0 && atomicCAS(&p.status->code, 0, TLC_DEV_INDEX) == 0) p.status->where = 402;
        pos = pos < 0 ? 0 : p.max_seq - 1;
    }
    const Visible vis(pos, p.window, p.keep);
    const int tiles = (vis.count + kKeys - 1) / kKeys, per = (tiles + nsplit - 1) / nsplit;
    const int t_lo = split * per < tiles ? split * per : tiles, t_hi = t_lo + per < tiles ? t_lo + per : tiles;
    bf16 *kbase = static_cast<bf16 *>(p.kc) + ((size_t)slot * p.max_seq * p.G + hk) * p.Dp;
    bf16 *vbase = static_cast<bf16 *>(p.vc) + ((size_t)slot * p.max_seq * p.G + hk) * p.Dp;
    const size_t key_stride = (size_t)p.G * p.Dp;
    const int newest = vis.count - 1;  // number of this step's own key: never read from the cache
    auto load_tile = [&](int tile, int stage) {
        for (int c = tid; c < kKeys * CH; c += kAttn) {
            const int key = c / CH, part = c % CH, v = tile * kKeys + key;
            const bool ok = v < newest && part * 8 < p.Dp;
            const size_t off = ok ? (size_t)vis.position(v) * key_stride + part * 8 : 0;
            cp_async16(ks + stage * TILE + key * PITCH + part * 8, kbase + off, ok);
            cp_async16(vs + stage * TILE + key * PITCH + part * 8, vbase + off, ok);
        }
        cp_async_commit();
    };
    // cache rows of earlier steps, norm weights and angles do not depend on the kernels in flight
    if (t_lo < t_hi) load_tile(t_lo, 0);
    constexpr int NP = D / 16;  // pair units of the 16 query rows per thread; one of the key
    const bool owner = newest / kKeys >= t_lo && newest / kKeys < t_hi;
    const bf16 *qn = static_cast<const bf16 *>(p.qn) + (size_t)(hk * grp + 16 * qt) * p.D;
    const bf16 *kn = static_cast<const bf16 *>(p.kn) + (size_t)hk * p.D;
    bf16 qw[NP][2], kw[2];
#pragma unroll
    for (int j = 0; j < NP; j++) {
        const int u = tid + kAttn * j, row = u / (D / 2);
        const Pair pr(u % (D / 2), p.rot);
        qw[j][0] = row < heads && pr.e0 < p.D ? qn[row * p.D + pr.e0] : from_f32<bf16>(0.f);
        qw[j][1] = row < heads && pr.e1 < p.D ? qn[row * p.D + pr.e1] : from_f32<bf16>(0.f);
    }
    const Pair kp(tid, p.rot);
    const bool kin = owner && tid < D / 2;
    kw[0] = kin && kp.e0 < p.D ? kn[kp.e0] : from_f32<bf16>(0.f);
    kw[1] = kin && kp.e1 < p.D ? kn[kp.e1] : from_f32<bf16>(0.f);
    for (int i = tid; i < half; i += kAttn) sincosf((float)pos * p.freq[i], &sn[i], &cs[i]);
    pdl_enter();

    const bf16 *q = static_cast<const bf16 *>(p.q) + (size_t)r * p.ldq, *kr = static_cast<const bf16 *>(p.k_raw) + (size_t)r * p.ldk;
    const bf16 *qg = q + (size_t)(hk * grp + 16 * qt) * p.D, *kg = kr + (size_t)hk * p.D;
    bf16 qv[NP][2], kv[2];
#pragma unroll
    for (int j = 0; j < NP; j++) {
        const int u = tid + kAttn * j, row = u / (D / 2);
        const Pair pr(u % (D / 2), p.rot);
        qv[j][0] = row < heads && pr.e0 < p.D ? qg[row * p.D + pr.e0] : from_f32<bf16>(0.f);
        qv[j][1] = row < heads && pr.e1 < p.D ? qg[row * p.D + pr.e1] : from_f32<bf16>(0.f);
    }
    kv[0] = kin && kp.e0 < p.D ? kg[kp.e0] : from_f32<bf16>(0.f);
    kv[1] = kin && kp.e1 < p.D ? kg[kp.e1] : from_f32<bf16>(0.f);
    auto squares = [&](const bf16 *x, int n) {  // rows are padded to whole pieces, with anything
        float s = 0.f;
        for (int i = tid; i < (n + 7) / 8; i += kAttn) {
            float f[8];
            unpack(__ldcg(reinterpret_cast<const uint4 *>(x) + i), f);
#pragma unroll
            for (int e = 0; e < 8; e++) s += 8 * i + e < n ? f[e] * f[e] : 0.f;
        }
        return s;
    };
    const float2 sq = block_sum2(squares(q, p.H * p.D), squares(kr, p.G * p.D), red);  // also the barrier behind cs / sn
    const float rq = 1.0f / sqrtf(sq.x / (float)(p.H * p.D) + p.eps), rk = 1.0f / sqrtf(sq.y / (float)(p.G * p.D) + p.eps);
    auto turn = [&](const Pair &pr, const bf16 (&v)[2], const bf16 (&w)[2], float scale, int i) {
        const float a = to_f32(v[0]) * scale * to_f32(w[0]), b = to_f32(v[1]) * scale * to_f32(w[1]);
        return pr.turn ? make_float2(a * cs[i] - b * sn[i], b * cs[i] + a * sn[i]) : make_float2(a, b);
    };
#pragma unroll
    for (int j = 0; j < NP; j++) {
        const int u = tid + kAttn * j, row = u / (D / 2), i = u % (D / 2);
        const Pair pr(i, p.rot);
        const float2 v = turn(pr, qv[j], qw[j], rq, i);
        qs[row * PITCH + pr.e0] = from_f32<bf16>(v.x);
        qs[row * PITCH + pr.e1] = from_f32<bf16>(v.y);
    }
    if (kin) {
        const float2 v = turn(kp, kv, kw, rk, tid);
        newk[kp.e0] = from_f32<bf16>(v.x);
        newk[kp.e1] = from_f32<bf16>(v.y);
        newv[kp.e0] = kv[0];
        newv[kp.e1] = kv[1];
        if (qt == 0) {
            bf16 *kd = kbase + (size_t)pos * key_stride, *vd = vbase + (size_t)pos * key_stride;
            if (kp.e0 < p.Dp) {
                kd[kp.e0] = newk[kp.e0];
                vd[kp.e0] = kv[0];
            }
            if (kp.e1 < p.Dp) {
                kd[kp.e1] = newk[kp.e1];
                vd[kp.e1] = kv[1];
            }
        }
    }
    __syncthreads();

    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    float o[NDT][4];
#pragma unroll
    for (int i = 0; i < NDT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const float scale2 = p.scale * 1.44269504088896340736f;
    const int mi = lane >> 3;
    for (int tile = t_lo; tile < t_hi; tile++) {
        const int stage = (tile - t_lo) & 1;
        if (tile + 1 < t_hi) {
            load_tile(tile + 1, stage ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        bf16 *kt = ks + stage * TILE, *vt = vs + stage * TILE;
        if (tile == newest / kKeys) {  // this step's own key and value
            for (int e = tid; e < D; e += kAttn) {
                kt[(newest % kKeys) * PITCH + e] = newk[e];
                vt[(newest % kKeys) * PITCH + e] = newv[e];
            }
            __syncthreads();
        }
        // each warp takes 16 keys
        float s[2][4] = {};
#pragma unroll
        for (int kk = 0; kk < KSTEPS; kk++) {
            uint32_t qa[4], kb[4];
            ldsm_x4(qa, qs + ((mi & 1) * 8 + (lane & 7)) * PITCH + 16 * kk + (mi >> 1) * 8);
            ldsm_x4(kb, kt + (16 * warp + (mi >> 1) * 8 + (lane & 7)) * PITCH + 16 * kk + (mi & 1) * 8);
            mma_bf16(s[0], qa, kb[0], kb[1]);
            mma_bf16(s[1], qa, kb[2], kb[3]);
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int v = tile * kKeys + 16 * warp + 8 * n + 2 * t + (e & 1);
                s[n][e] = v < vis.count ? s[n][e] * scale2 : -INFINITY;
                mx[e >> 1] = fmaxf(mx[e >> 1], s[n][e]);
            }
        float corr[2];
#pragma unroll
        for (int h = 0; h < 2; h++) {
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
            const float m_new = fmaxf(m_run[h], mx[h]), base = m_new == -INFINITY ? 0.f : m_new;
            corr[h] = exp2f(m_run[h] - base);
            m_run[h] = m_new;
            float sum = 0.f;
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    s[n][2 * h + e] = exp2f(s[n][2 * h + e] - base);
                    sum += s[n][2 * h + e];
                }
            l_run[h] = l_run[h] * corr[h] + sum;
        }
#pragma unroll
        for (int d = 0; d < NDT; d++) {
            o[d][0] *= corr[0];
            o[d][1] *= corr[0];
            o[d][2] *= corr[1];
            o[d][3] *= corr[1];
        }
        uint32_t hi[4], lo[4];
        split_pair(s[0][0], s[0][1], hi[0], lo[0]);
        split_pair(s[0][2], s[0][3], hi[1], lo[1]);
        split_pair(s[1][0], s[1][1], hi[2], lo[2]);
        split_pair(s[1][2], s[1][3], hi[3], lo[3]);
#pragma unroll
        for (int jd = 0; jd < KSTEPS; jd++) {
            uint32_t b[4];
            ldsm_x4_trans(b, vt + (16 * warp + (mi & 1) * 8 + (lane & 7)) * PITCH + 16 * jd + (mi >> 1) * 8);
            mma_bf16(o[2 * jd], hi, b[0], b[1]);
            mma_bf16(o[2 * jd + 1], hi, b[2], b[3]);
            mma_bf16(o[2 * jd], lo, b[0], b[1]);
            mma_bf16(o[2 * jd + 1], lo, b[2], b[3]);
        }
        __syncthreads();
    }
    // the four warps' results meet in the tile area: [4][16][D]
    float *ow = reinterpret_cast<float *>(smem_raw);
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
        if (t == 0) {
            sm_m[warp][g + 8 * h] = m_run[h];
            sm_l[warp][g + 8 * h] = l_run[h];
        }
#pragma unroll
        for (int d = 0; d < NDT; d++) {
            ow[(size_t)(warp * 16 + g + 8 * h) * D + 8 * d + 2 * t] = o[d][2 * h];
            ow[(size_t)(warp * 16 + g + 8 * h) * D + 8 * d + 2 * t + 1] = o[d][2 * h + 1];
        }
    }
    __syncthreads();
    const int cols = D / nsplit, stride = cols + 4;
    const uint32_t merge_addr = (uint32_t)__cvta_generic_to_shared(merge);
    if (cluster) asm volatile("barrier.cluster.wait.aligned;" ::: "memory");  // every peer is running
    for (int i = tid; i < heads * (D / 4); i += kAttn) {
        const int row = i / (D / 4), e = 4 * (i % (D / 4));
        const float m = fmaxf(fmaxf(sm_m[0][row], sm_m[1][row]), fmaxf(sm_m[2][row], sm_m[3][row]));
        const float base = m == -INFINITY ? 0.f : m;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        float l = 0.f;
#pragma unroll
        for (int w = 0; w < 4; w++) {
            const float f = exp2f(sm_m[w][row] - base);
            const float4 v = *reinterpret_cast<const float4 *>(ow + (size_t)(w * 16 + row) * D + e);
            a.x += f * v.x;
            a.y += f * v.y;
            a.z += f * v.z;
            a.w += f * v.w;
            l += f * sm_l[w][row];
        }
        const int dst = e / cols, c = e - dst * cols, at = (split * 16 + row) * stride;
        if (cluster) {
            const uint32_t to = remote_address(merge_addr + 4 * at, dst);
            store_remote(to + 4 * c, a);
            if (c == 0) store_remote(to + 4 * cols, make_float2(m, l));
        } else {
            *reinterpret_cast<float4 *>(merge + at + c) = a;
            if (c == 0) *reinterpret_cast<float2 *>(merge + at + cols) = make_float2(m, l);
        }
    }
    if (cluster) {
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    } else {
        __syncthreads();
    }
    for (int i = tid; i < heads * cols; i += kAttn) {
        const int row = i / cols, c = i % cols, e = split * cols + c;
        float m = -INFINITY;
        for (int s = 0; s < nsplit; s++) m = fmaxf(m, merge[(s * 16 + row) * stride + cols]);
        const float base = m == -INFINITY ? 0.f : m;
        float a = 0.f, l = 0.f;
        for (int s = 0; s < nsplit; s++) {
            const float *mr = merge + (size_t)(s * 16 + row) * stride;
            const float f = exp2f(mr[cols] - base);
            a += f * mr[c];
            l += f * mr[cols + 1];
        }
        if (e < p.D)
            static_cast<bf16 *>(p.out)[(size_t)r * p.ldo + (size_t)(hk * grp + 16 * qt + row) * p.D + e] =
                from_f32<bf16>(l > 0.f ? a / l : 0.f);
    }
}

constexpr int kRowsMaxD = 512;

// One warp per (row, query head): 32 keys at a time, a key per lane for the scores, a stretch of
// columns per lane for the weighted sum.
template <typename T>
__global__ void __launch_bounds__(128) window_rows_kernel(const WindowAttn p) {
    extern __shared__ float qsm[];  // [4][Dp]
    pdl_enter();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long w = (long long)blockIdx.x * 4 + warp;
    if (w >= (long long)p.m * p.H) return;
    const int r = (int)(w / p.H), head = (int)(w % p.H), hk = head / (p.H / p.G);
    float *q = qsm + warp * p.Dp;
    const T *qg = static_cast<const T *>(p.q) + ((size_t)r * p.H + head) * p.Dp;
    for (int e = lane; e < p.Dp; e += 32) q[e] = to_f32(qg[e]);
    __syncwarp();
    int pos = p.pos[r];
    if (pos < 0 || pos >= p.max_seq) {
        if (lane == 0 && atomicCAS(&p.status->code, 0, TLC_DEV_INDEX) == 0) p.status->where = 403;
        pos = pos < 0 ? 0 : p.max_seq - 1;
    }
    const Visible vis(pos, p.window, p.keep);
    const size_t base = ((size_t)p.slot[r] * p.max_seq * p.G + hk) * p.Dp, stride = (size_t)p.G * p.Dp;
    const T *kc = static_cast<const T *>(p.kc) + base, *vc = static_cast<const T *>(p.vc) + base;
    float acc[kRowsMaxD / 32];
#pragma unroll
    for (int i = 0; i < kRowsMaxD / 32; i++) acc[i] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;
    for (int v0 = 0; v0 < vis.count; v0 += 32) {
        const int v = v0 + lane;
        const int at = v < vis.count ? vis.position(v) : 0;
        float s = -INFINITY;
        if (v < vis.count) {
            const uint4 *k = reinterpret_cast<const uint4 *>(kc + (size_t)at * stride);
            s = 0.f;
            for (int c = 0; c < p.Dp / Vec<T>::N; c++) {
                float f[Vec<T>::N];
                unpack(k[c], f);
#pragma unroll
                for (int e = 0; e < Vec<T>::N; e++) s = fmaf(f[e], q[c * Vec<T>::N + e], s);
            }
            s *= p.scale;
        }
        float mx = s;
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        const float m_new = fmaxf(m_run, mx), corr = expf(m_run - m_new);
        const float pr = expf(s - m_new);
        l_run = l_run * corr + warp_sum(pr);
        m_run = m_new;
#pragma unroll
        for (int i = 0; i < kRowsMaxD / 32; i++) acc[i] *= corr;
        const int n = vis.count - v0 < 32 ? vis.count - v0 : 32;
        for (int j = 0; j < n; j++) {
            const float pj = __shfl_sync(0xffffffffu, pr, j);
            const T *val = vc + (size_t)__shfl_sync(0xffffffffu, at, j) * stride;
#pragma unroll
            for (int i = 0; i < kRowsMaxD / 32; i++)
                if (32 * i + lane < p.D) acc[i] = fmaf(pj, to_f32(val[32 * i + lane]), acc[i]);
        }
    }
    T *out = static_cast<T *>(p.out) + (size_t)r * p.ldo + (size_t)head * p.D;
#pragma unroll
    for (int i = 0; i < kRowsMaxD / 32; i++)
        if (32 * i + lane < p.D) out[32 * i + lane] = from_f32<T>(acc[i] / l_run);
}

template <int D>
int32_t prefill_t(tlc_ctx *ctx, const WindowAttn &p, int slot) {
    const size_t smem = (size_t)(4 * kKeys + 64) * (D + 8) * 2;
    static bool done[64] = {};
    if (!done[ctx->device & 63]) {
        TLC_CUDA(cudaFuncSetAttribute(window_prefill_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        TLC_CUDA(cudaFuncSetAttribute(window_prefill_kernel<D>, cudaFuncAttributePreferredSharedMemoryCarveout,
                                      cudaSharedmemCarveoutMaxShared));
        done[ctx->device & 63] = true;
    }
    const int rows = p.m * (p.H / p.G);
    cudaError_t le = tlc_launch_pdl(ctx, window_prefill_kernel<D>, dim3((rows + 63) / 64, p.G), dim3(kAttn), smem, p, slot);
    if (le != cudaSuccess) {
        cudaGetLastError();
        return tlc_fail(TLC_ERR_CUDA, "window attention launch failed: %s", cudaGetErrorString(le));
    }
    TLC_CHECK_LAUNCH(ctx);
    return TLC_OK;
}

template <int D>
int32_t decode_t(tlc_ctx *ctx, const WindowAttn &p) {
    static bool done[64] = {};
    if (!done[ctx->device & 63]) {
        TLC_CUDA(cudaFuncSetAttribute(window_decode_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                      (int)decode_smem(D, 8, D)));
        TLC_CUDA(cudaFuncSetAttribute(window_decode_kernel<D>, cudaFuncAttributePreferredSharedMemoryCarveout,
                                      cudaSharedmemCarveoutMaxShared));
        done[ctx->device & 63] = true;
    }
    const int grp = p.H / p.G;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)(p.nsplit * ((grp + 15) / 16)), (unsigned)p.G, (unsigned)p.m);
    cfg.blockDim = dim3(kAttn);
    cfg.dynamicSmemBytes = decode_smem(D, p.nsplit, p.rot / 2);
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (ctx->use_pdl && ctx->pdl_small) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (p.nsplit > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = (unsigned)p.nsplit;
        attr[n].val.clusterDim.y = 1;
        attr[n++].val.clusterDim.z = 1;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    cudaError_t le = cudaLaunchKernelEx(&cfg, window_decode_kernel<D>, p);
    if (le != cudaSuccess) {
        cudaGetLastError();
        return tlc_fail(TLC_ERR_CUDA, "window attention launch failed: %s", cudaGetErrorString(le));
    }
    TLC_CHECK_LAUNCH(ctx);
    return TLC_OK;
}

}  // namespace

bool window_tensor_cores(int D) { return D <= 256; }

int32_t launch_window_prefill(tlc_ctx *ctx, const WindowAttn &p, int slot) {
    if (p.D <= 32) return prefill_t<32>(ctx, p, slot);
    if (p.D <= 64) return prefill_t<64>(ctx, p, slot);
    if (p.D <= 96) return prefill_t<96>(ctx, p, slot);
    if (p.D <= 128) return prefill_t<128>(ctx, p, slot);
    if (p.D <= 192) return prefill_t<192>(ctx, p, slot);
    return prefill_t<256>(ctx, p, slot);
}

int32_t launch_window_decode(tlc_ctx *ctx, WindowAttn p) {
    // splits: enough CTAs for the SMs, at most eight (a portable cluster), no more than tiles
    const long long reach = (long long)p.window + p.keep;
    const int most = reach < p.max_seq ? (int)reach : p.max_seq;
    const int tiles = (most + kKeys - 1) / kKeys;
    p.nsplit = 1;
    while (p.nsplit < 8 && 2 * p.nsplit <= tiles) p.nsplit *= 2;
    if (p.D <= 32) return decode_t<32>(ctx, p);
    if (p.D <= 64) return decode_t<64>(ctx, p);
    if (p.D <= 96) return decode_t<96>(ctx, p);
    if (p.D <= 128) return decode_t<128>(ctx, p);
    if (p.D <= 192) return decode_t<192>(ctx, p);
    return decode_t<256>(ctx, p);
}

template <typename T>
int32_t launch_window_rows(tlc_ctx *ctx, const WindowAttn &p) {
    TLC_REQUIRE(p.D <= kRowsMaxD, TLC_ERR_INVALID_OPERATION, "attention: heads of %d values (at most %d)", p.D, kRowsMaxD);
    const long long warps = (long long)p.m * p.H;
    cudaError_t le = tlc_launch_pdl(ctx, window_rows_kernel<T>, dim3((unsigned)((warps + 3) / 4)), dim3(128),
                                    (size_t)4 * p.Dp * sizeof(float), p);
    if (le != cudaSuccess) {
        cudaGetLastError();
        return tlc_fail(TLC_ERR_CUDA, "window attention launch failed: %s", cudaGetErrorString(le));
    }
    TLC_CHECK_LAUNCH(ctx);
    return TLC_OK;
}
template int32_t launch_window_rows<bf16>(tlc_ctx *, const WindowAttn &);
template int32_t launch_window_rows<float>(tlc_ctx *, const WindowAttn &);

}  // namespace tlc_dense
