// Many activation rows against dense weights: y = epilogue(x . W^T) for several weights, gate/up
// pairs and families of experts in ONE launch.
//
// bf16: persistent tcgen05 kernel.  A tile is 128 activation rows x 256 weight rows (a pair: 128
// gate rows and the matching 128 up rows); both operands arrive by TMA in 64-wide K steps with the
// 128-byte swizzle, four stages of 48 KB; one thread issues tcgen05.mma (M = 128, N = 256, K = 16)
// into one of two 256-column accumulators in tensor memory, eight warps drain the other one
// meanwhile.  Two stretches of K (attention output and feed-forward down) may add up in one
// accumulator.  The tiles of a family of experts come from the row offsets the router left in
// device memory.
// f32: the same tiles of work, 64 x 64, on the FMA pipes; no reduced-precision product anywhere.
#include <cudaTypedefs.h>

#include "tlc_dense.cuh"
#include "tlc_gemm_kernel.cuh"

namespace tlc_dense {

using namespace tlc_gemm;

namespace {

constexpr int kStagesD = 4;
constexpr int kABytes = 128 * 128, kBBytes = 256 * 128, kStageBytesD = kABytes + kBBytes;
constexpr int kEpilogueWarps = 8;  // two per lane quarter of the tensor memory, taking the column pieces in turn
constexpr int kThreadsD = 32 * (2 + kEpilogueWarps);  // and the TMA warp, the MMA warp
constexpr size_t kSmemD = 1024 + (size_t)kStagesD * kStageBytesD + 256 + (size_t)(2 * kMaxSlots + 4) * sizeof(int);
constexpr int kTurnPitch = 20;  // floats per row of an epilogue warp's turning area: 32 rows of 16 columns
constexpr size_t kSmemTurn = (size_t)kEpilogueWarps * 32 * kTurnPitch * sizeof(float);
static_assert(((2 * kMaxSlots + 4) * sizeof(int)) % 16 == 0, "the turning area starts on a 16-byte boundary");

// Instruction descriptor: bf16 x bf16 -> f32, both operands K-major, M = 128, N = 256.
constexpr uint32_t kIdescBf16 = idesc_for(256) | (1u << 7) | (1u << 10);

struct Tile {
    int group, expert;  // expert: weight of a family, else 0
    int row0, rows;     // first row of A / out, rows that exist in this tile
    int n0;
};

// Slots are the dense groups and the single experts, in order; start[s] is the first tile of slot s
// (start[slots]: all tiles), row0[s] the first row of an expert's slot.  Call with all threads.
template <int BM, int BN>
__device__ void plan_tiles(const GemmParams &p, int *start, int *first_row) {
    const int tid = threadIdx.x;
    // tiles of each slot
    int base = 0;
    for (int g = 0; g < p.n_groups; g++) {
        const GemmGroup &gr = p.g[g];
        const int bn = gr.epi >= EPI_CLAMPED_GLU ? (BN == 256 ? 128 : BN) : BN;
        const int nt = (gr.n + bn - 1) / bn, slots = gr.experts > 0 ? gr.experts : 1;
        for (int e = tid; e < slots; e += blockDim.x) {
            const int lo = gr.experts > 0 ? __ldcg(gr.off + e) : 0;
            const int rows = gr.experts > 0 ? __ldcg(gr.off + e + 1) - lo : gr.rows;
            start[base + e] = (rows + BM - 1) / BM * nt;
            first_row[base + e] = lo;
        }
        base += slots;
    }
    __syncthreads();
    if (tid < 32) {  // exclusive sums, 32 slots at a time
        int carry = 0;
        for (int s0 = 0; s0 < base; s0 += 32) {
            const int s = s0 + tid;
            const int c = s < base ? start[s] : 0;
            int incl = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int t = __shfl_up_sync(0xffffffffu, incl, o);
                if (tid >= o) incl += t;
            }
            if (s < base) start[s] = carry + incl - c;
            carry += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (tid == 0) start[base] = carry;
    }
    __syncthreads();
}

// Tile t; `slot` only moves forward (tiles are asked for in increasing order).
template <int BM, int BN>
__device__ __forceinline__ Tile tile_at(const GemmParams &p, const int *start, const int *first_row, int t, int &slot) {
    while (t >= start[slot + 1]) slot++;
    Tile r;
    int g = 0, base = 0;
    for (;;) {
        const int slots = p.g[g].experts > 0 ? p.g[g].experts : 1;
        if (slot < base + slots) break;
        base += slots;
        g++;
    }
    r.group = g;
    r.expert = slot - base;
    const GemmGroup &gr = p.g[g];
    const int lo = first_row[slot];
    const int rows = gr.experts > 0 ? __ldcg(gr.off + r.expert + 1) - lo : gr.rows;
    const int mt = (rows + BM - 1) / BM, local = t - start[slot];
    const int m = local % mt, n = local / mt;  // row tiles fastest: a weight tile is shared by neighbours
    r.row0 = lo + m * BM;
    r.rows = rows - m * BM < BM ? rows - m * BM : BM;
    const int bn = gr.epi >= EPI_CLAMPED_GLU ? (BN == 256 ? 128 : BN) : BN;
    r.n0 = n * bn;
    return r;
}

// 32 consecutive outputs of one row.  `up`: the pair's second sums.
__device__ __forceinline__ void store_piece(const GemmGroup &g, const uint32_t (&acc)[32], const uint32_t (&up)[32], int row,
                                            int nb) {
    const bool whole = nb + 32 <= g.n;
    if (g.epi == EPI_ADD_F32 || g.epi == EPI_STORE_F32 || g.epi == EPI_SOFTCAP_F32) {
        float *out = static_cast<float *>(g.out) + (size_t)row * g.ldo + nb;
        const bool add = g.epi == EPI_ADD_F32;
        if (whole && (g.ldo & 3) == 0) {
#pragma unroll
            for (int v = 0; v < 8; v++) {
                float4 o = add ? __ldcg(reinterpret_cast<const float4 *>(out + 4 * v)) : make_float4(0.f, 0.f, 0.f, 0.f);
                float b[4] = {0.f, 0.f, 0.f, 0.f};
                if (g.bias)
#pragma unroll
                    for (int e = 0; e < 4; e++) b[e] = to_f32(static_cast<const bf16 *>(g.bias)[nb + 4 * v + e]);
                o.x += __uint_as_float(acc[4 * v]) + b[0];
                o.y += __uint_as_float(acc[4 * v + 1]) + b[1];
                o.z += __uint_as_float(acc[4 * v + 2]) + b[2];
                o.w += __uint_as_float(acc[4 * v + 3]) + b[3];
                if (g.epi == EPI_SOFTCAP_F32) {
                    o.x = g.limit * tanhf(o.x / g.limit);
                    o.y = g.limit * tanhf(o.y / g.limit);
                    o.z = g.limit * tanhf(o.z / g.limit);
                    o.w = g.limit * tanhf(o.w / g.limit);
                }
                *reinterpret_cast<float4 *>(out + 4 * v) = o;
            }
        } else {
#pragma unroll
            for (int e = 0; e < 32; e++)
                if (nb + e < g.n) {
                    const float v = (add ? out[e] : 0.f) + __uint_as_float(acc[e]) +
                                    (g.bias ? to_f32(static_cast<const bf16 *>(g.bias)[nb + e]) : 0.f);
                    out[e] = g.epi == EPI_SOFTCAP_F32 ? g.limit * tanhf(v / g.limit) : v;
                }
        }
        return;
    }
    __align__(16) bf16 h[32];
    if (g.epi == EPI_STORE) {
#pragma unroll
        for (int e = 0; e < 32; e++) {
            float v = __uint_as_float(acc[e]);
            if (g.bias && (whole || nb + e < g.n)) v += to_f32(static_cast<const bf16 *>(g.bias)[nb + e]);
            h[e] = from_f32<bf16>(v);
        }
    } else {
        const float si = g.in_scale ? g.in_scale[row] : 1.f;
        const float so = g.out_scale ? sigmoid_f(g.out_scale[(size_t)row * g.out_scale_stride]) : 1.f;
        if (g.epi == EPI_CLAMPED_GLU) {
#pragma unroll
            for (int e = 0; e < 32; e++)
                h[e] = from_f32<bf16>(clamped_glu(si * __uint_as_float(acc[e]), si * __uint_as_float(up[e]), g.limit) * so);
        } else {
#pragma unroll
            for (int e = 0; e < 32; e++) {
                float gate = si * __uint_as_float(acc[e]), u = si * __uint_as_float(up[e]);
                if (g.bias && (whole || nb + e < g.n)) {
                    gate += to_f32(static_cast<const bf16 *>(g.bias)[nb + e]);
                    u += to_f32(static_cast<const bf16 *>(g.bias2)[nb + e]);
                }
                h[e] = from_f32<bf16>(silu_mul(gate, u) * so);
            }
        }
    }
    bf16 *out = static_cast<bf16 *>(g.out) + (size_t)row * g.ldo + nb;
    if (whole && (g.ldo & 7) == 0) {
#pragma unroll
        for (int v = 0; v < 4; v++) *reinterpret_cast<uint4 *>(out + 8 * v) = *reinterpret_cast<const uint4 *>(h + 8 * v);
    } else {
#pragma unroll
        for (int e = 0; e < 32; e++)
            if (nb + e < g.n) out[e] = h[e];
    }
}

// 32 columns of the warp's 32 rows (lane = row of `acc`) into the residual streams.  Rows turn into
// columns through shared memory, 16 columns at a time, so that four lanes share a row's 64 bytes and
// the loads of all streams are in flight together.  Rows from `rows` on (if below 32) do not exist.
template <int MAXS>
__device__ __forceinline__ void store_streams(const GemmGroup &g, const StreamsOut &st, const uint32_t (&acc)[32], float *turn,
                                              int row0, int rows, int nb, int lane) {
#pragma unroll
    for (int half = 0; half < 2; half++) {
        if (nb + 16 * half >= g.n) break;
        __syncwarp();
#pragma unroll
        for (int v = 0; v < 4; v++)
            *reinterpret_cast<float4 *>(turn + lane * kTurnPitch + 4 * v) =
                make_float4(__uint_as_float(acc[16 * half + 4 * v]), __uint_as_float(acc[16 * half + 4 * v + 1]),
                            __uint_as_float(acc[16 * half + 4 * v + 2]), __uint_as_float(acc[16 * half + 4 * v + 3]));
        __syncwarp();
        const int n = nb + 16 * half + 4 * (lane & 3);
        if (n >= g.n) continue;
        if ((g.n & 3) != 0) {  // rows do not start on 16-byte boundaries
            for (int i = lane >> 2; i < rows && i < 32; i += 8)
                for (int e = 0; e < 4 && n + e < g.n; e++)
                    streams_column<bf16>(st, row0 + i, g.n, n + e,
                                         turn[i * kTurnPitch + 4 * (lane & 3) + e] +
                                             (g.bias ? to_f32(static_cast<const bf16 *>(g.bias)[n + e]) : 0.f));
            continue;
        }
        auto four = [&](const void *p, float (&f)[4]) {
            const uint2 v = __ldg(reinterpret_cast<const uint2 *>(static_cast<const bf16 *>(p) + n));
            f[0] = __uint_as_float(v.x << 16);
            f[1] = __uint_as_float(v.x & 0xffff0000u);
            f[2] = __uint_as_float(v.y << 16);
            f[3] = __uint_as_float(v.y & 0xffff0000u);
        };
        float bias[4] = {0.f, 0.f, 0.f, 0.f}, scale[4], w[4], b[4];
        if (g.bias) four(g.bias, bias);
        four(st.scale, scale);
        if (st.h) {
            four(st.w, w);
            four(st.b, b);
        }
        constexpr int AT_ONCE = MAXS > 4 ? 2 : 4;
#pragma unroll
        for (int i0 = 0; i0 < 4; i0 += AT_ONCE) {
            float4 x[AT_ONCE][MAXS];
#pragma unroll
            for (int i = 0; i < AT_ONCE; i++) {
                const int r = 8 * (i0 + i) + (lane >> 2);
#pragma unroll
                for (int s = 0; s < MAXS; s++)
                    if (s < stream_count<MAXS>(st) && r < rows)
                        x[i][s] = __ldcg(reinterpret_cast<const float4 *>(st.x + s * st.plane + (int64_t)(row0 + r) * g.n + n));
            }
#pragma unroll
            for (int i = 0; i < AT_ONCE; i++) {
                const int r = 8 * (i0 + i) + (lane >> 2);
                if (r >= rows) continue;
                const float4 a = *reinterpret_cast<const float4 *>(turn + r * kTurnPitch + 4 * (lane & 3));
                const float av[4] = {a.x, a.y, a.z, a.w};
                float h[4];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    float xs[MAXS];
#pragma unroll
                    for (int s = 0; s < MAXS; s++) xs[s] = e == 0 ? x[i][s].x : e == 1 ? x[i][s].y : e == 2 ? x[i][s].z : x[i][s].w;
                    const float u = update_streams(st, (av[e] + bias[e]) * scale[e], xs);
#pragma unroll
                    for (int s = 0; s < MAXS; s++) {
                        if (e == 0) x[i][s].x = xs[s];
                        if (e == 1) x[i][s].y = xs[s];
                        if (e == 2) x[i][s].z = xs[s];
                        if (e == 3) x[i][s].w = xs[s];
                    }
                    h[e] = st.h ? tanh_norm(u, st.alpha, w[e], b[e]) : 0.f;
                }
#pragma unroll
                for (int s = 0; s < MAXS; s++)
                    if (s < stream_count<MAXS>(st)) *reinterpret_cast<float4 *>(st.x + s * st.plane + (int64_t)(row0 + r) * g.n + n) = x[i][s];
                if (st.h) {
                    const __nv_bfloat162 lo = __floats2bfloat162_rn(h[0], h[1]), hi = __floats2bfloat162_rn(h[2], h[3]);
                    *reinterpret_cast<uint2 *>(static_cast<bf16 *>(st.h) + (int64_t)(row0 + r) * st.ldh + n) =
                        make_uint2(*reinterpret_cast<const uint32_t *>(&lo), *reinterpret_cast<const uint32_t *>(&hi));
                }
            }
        }
    }
}

// MAXS > 0: the form whose group ends in EPI_STREAMS, for MAXS streams (8: for up to so many).
template <int MAXS>
__global__ void __launch_bounds__(kThreadsD, 1) dense_gemm_kernel(const __grid_constant__ GemmParams p) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *tiles = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint64_t *full = reinterpret_cast<uint64_t *>(tiles + (size_t)kStagesD * kStageBytesD);
    uint64_t *empty = full + kStagesD, *acc_full = empty + kStagesD, *acc_empty = acc_full + 2;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(acc_empty + 2);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
    int *start = reinterpret_cast<int *>(reinterpret_cast<uint8_t *>(full) + 256);
    int *first_row = start + kMaxSlots + 2;
    [[maybe_unused]] float *turning = reinterpret_cast<float *>(first_row + kMaxSlots + 2);

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (int s = 0; s < kStagesD; s++) {
            mbar_init(&full[s], 1);
            mbar_init(&empty[s], 1);
        }
        for (int a = 0; a < 2; a++) {
            mbar_init(&acc_full[a], 1);
            mbar_init(&acc_empty[a], kEpilogueWarps);
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(512u)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    pdl_enter();
    plan_tiles<128, 256>(p, start, first_row);
    const int n_tiles = start[p.slots];

    if (warp == 0) {
        if (lane == 0) {
            int slot = 0, j = 0;
            bool alive = true;
            for (int t = blockIdx.x; alive && t < n_tiles; t += gridDim.x) {
                const Tile tl = tile_at<128, 256>(p, start, first_row, t, slot);
                const GemmGroup &g = p.g[tl.group];
                for (int seg = 0; alive && seg < 2; seg++) {
                    const int steps = (g.k[seg] + kBK - 1) / kBK;
                    const CUtensorMap *am = p.maps + g.a_map[seg];
                    const CUtensorMap *bm = p.maps + g.b_map[seg] + (size_t)tl.expert * g.map_stride;
                    const CUtensorMap *um = g.b2_map >= 0 ? p.maps + g.b2_map + (size_t)tl.expert * g.map_stride : bm;
                    const int first = g.b_row0 + tl.n0, second = g.b2_map >= 0 ? first : first + 128;  // rows of the tile's halves
                    for (int s = 0; s < steps; s++, j++) {
                        const int st = j % kStagesD;
                        if (!mbar_wait(&empty[st], ((j / kStagesD) & 1u) ^ 1u, abort_flag, p.status, 21, p.wait_ns)) {
                            alive = false;
                            break;
                        }
                        const uint32_t bar = smem_u32(&full[st]);
                        const uint32_t at = smem_u32(tiles + (size_t)st * kStageBytesD);
                        mbar_arrive_expect_tx(&full[st], kStageBytesD);
                        tma_load_2d(at, am, s * kBK, g.a_row0 + tl.row0, bar);
                        tma_load_2d(at + kABytes, bm, s * kBK, first, bar);
                        tma_load_2d(at + kABytes + 128 * 128, um, s * kBK, second, bar);
                    }
                }
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        int slot = 0, j = 0, it = 0;
        for (int t = blockIdx.x; t < n_tiles; t += gridDim.x, it++) {
            const Tile tl = tile_at<128, 256>(p, start, first_row, t, slot);
            const GemmGroup &g = p.g[tl.group];
            const int steps = (g.k[0] + kBK - 1) / kBK + (g.k[1] + kBK - 1) / kBK;
            const int a = it & 1;
            const bool free_acc =
                __all_sync(0xffffffffu, mbar_wait(&acc_empty[a], ((it >> 1) & 1u) ^ 1u, abort_flag, p.status, 22, p.wait_ns));
            tc_fence_after();
            for (int s = 0; s < steps; s++, j++) {
                const int st = j % kStagesD;
                const bool ready = __all_sync(0xffffffffu, mbar_wait(&full[st], (j / kStagesD) & 1u, abort_flag, p.status, 23, p.wait_ns));
                tc_fence_after();
                if (lane == 0 && ready && free_acc) {
                    const uint32_t aa = smem_u32(tiles + (size_t)st * kStageBytesD), bb = aa + kABytes;
#pragma unroll
                    for (int k16 = 0; k16 < kBK / 16; k16++)
                        umma_f16(tmem + 256 * a, make_desc(aa + k16 * 32), make_desc(bb + k16 * 32), kIdescBf16,
                                 (s > 0 || k16 > 0) ? 1u : 0u);
                }
                if (lane == 0) umma_commit(&empty[st]);
                __syncwarp();
            }
            if (lane == 0) umma_commit(&acc_full[a]);
            __syncwarp();
        }
    } else {
        const int wq = warp & 3, turn = (warp - 2) >> 2;  // tensor-memory lanes this warp may read: 32 wq ..
        int slot = 0, it = 0;
        for (int t = blockIdx.x; t < n_tiles; t += gridDim.x, it++) {
            const Tile tl = tile_at<128, 256>(p, start, first_row, t, slot);
            const GemmGroup &g = p.g[tl.group];
            const int a = it & 1;
            if constexpr (MAXS > 0) {  // the old streams on their way to the L2 while the tile's products run
                if ((g.n & 3) == 0)
                    for (int i = tid - 64; i < tl.rows * p.st.n; i += 32 * kEpilogueWarps) {
                        const int s = i / tl.rows, n = g.n - tl.n0 < 256 ? g.n - tl.n0 : 256;
                        prefetch_l2(p.st.x + s * p.st.plane + (int64_t)(tl.row0 + i - s * tl.rows) * g.n + tl.n0, (uint32_t)n * 4);
                    }
            }
            const bool done = mbar_wait(&acc_full[a], (it >> 1) & 1u, abort_flag, p.status, 24, p.wait_ns);
            tc_fence_after();
            const int row = 32 * wq + lane;
            const bool pair = g.epi >= EPI_CLAMPED_GLU;
            const int pieces = pair ? 4 : 8;
#pragma unroll 1
            for (int c = turn; c < pieces; c += kEpilogueWarps / 4) {
                if (tl.n0 + 32 * c >= g.n) break;
                uint32_t r[32], u[32];
                const uint32_t at = tmem + ((uint32_t)(32 * wq) << 16) + 256 * a + 32 * c;
                tmem_ld32(at, r);
                if (pair) tmem_ld32(at + 128, u);
                if constexpr (MAXS > 0) {
                    if (done && g.epi == EPI_STREAMS)
                        store_streams<MAXS>(g, p.st, r, turning + (warp - 2) * 32 * kTurnPitch, tl.row0 + 32 * wq, tl.rows - 32 * wq,
                                            tl.n0 + 32 * c, lane);
                } else {
                    if (done && row < tl.rows) store_piece(g, r, u, tl.row0 + row, tl.n0 + 32 * c);
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[a]);
        }
    }
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
    }
}

// f32: 64 x 64 outputs per tile and 256 threads, 4 x 4 outputs per thread, K in steps of 16.
__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const __grid_constant__ GemmParams p) {
    __shared__ float as[16][68], bs[16][68], us[16][68];
    __shared__ int start[kMaxSlots + 2], first_row[kMaxSlots + 2];
    pdl_enter();
    plan_tiles<64, 64>(p, start, first_row);
    const int n_tiles = start[p.slots], tid = threadIdx.x;
    const int tr = tid / 16, tc = tid % 16;
    int slot = 0;
    for (int t = blockIdx.x; t < n_tiles; t += gridDim.x) {
        const Tile tl = tile_at<64, 64>(p, start, first_row, t, slot);
        const GemmGroup &g = p.g[tl.group];
        const bool pair = g.epi >= EPI_CLAMPED_GLU;
        float acc[4][4] = {}, acu[4][4] = {};
        for (int seg = 0; seg < 2 && g.k[seg] > 0; seg++) {
            const float *a = static_cast<const float *>(g.a[seg]);
            const float *b = static_cast<const float *>(g.experts > 0 ? g.b_tab[tl.expert] : g.b[seg]);
            const float *u = static_cast<const float *>(!pair ? nullptr : g.experts > 0 ? g.b2_tab[tl.expert] : g.b2);
            for (int k0 = 0; k0 < g.k[seg]; k0 += 16) {
                __syncthreads();
                for (int i = tid; i < 64 * 16; i += 256) {
                    const int r = i / 16, k = i % 16;
                    const bool kin = k0 + k < g.k[seg];
                    as[k][r] = kin && r < tl.rows ? a[(size_t)(tl.row0 + r) * g.lda[seg] + k0 + k] : 0.f;
                    const bool nin = kin && tl.n0 + r < g.n;
                    bs[k][r] = nin ? b[(size_t)(tl.n0 + r) * g.ldb[seg] + k0 + k] : 0.f;
                    if (pair) us[k][r] = nin ? u[(size_t)(tl.n0 + r) * g.ldb[seg] + k0 + k] : 0.f;
                }
                __syncthreads();
#pragma unroll
                for (int k = 0; k < 16; k++) {
                    const float4 av = *reinterpret_cast<const float4 *>(&as[k][4 * tr]);
                    const float4 bv = *reinterpret_cast<const float4 *>(&bs[k][4 * tc]);
                    const float ar[4] = {av.x, av.y, av.z, av.w}, br[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
                    for (int i = 0; i < 4; i++)
#pragma unroll
                        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(ar[i], br[j], acc[i][j]);
                    if (pair) {
                        const float4 uv = *reinterpret_cast<const float4 *>(&us[k][4 * tc]);
                        const float ur[4] = {uv.x, uv.y, uv.z, uv.w};
#pragma unroll
                        for (int i = 0; i < 4; i++)
#pragma unroll
                            for (int j = 0; j < 4; j++) acu[i][j] = fmaf(ar[i], ur[j], acu[i][j]);
                    }
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int r = 4 * tr + i, row = tl.row0 + r;
            if (r >= tl.rows) continue;
            const float si = pair && g.in_scale ? g.in_scale[row] : 1.f;
            const float so = pair && g.out_scale ? sigmoid_f(g.out_scale[(size_t)row * g.out_scale_stride]) : 1.f;
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int n = tl.n0 + 4 * tc + j;
                if (n >= g.n) continue;
                float *out = static_cast<float *>(g.out) + (size_t)row * g.ldo + n;
                float v = acc[i][j];
                if (pair) {
                    float gate = si * v, up = si * acu[i][j];
                    if (g.bias) gate += static_cast<const float *>(g.bias)[n];
                    if (g.bias2) up += static_cast<const float *>(g.bias2)[n];
                    v = (g.epi == EPI_CLAMPED_GLU ? clamped_glu(gate, up, g.limit) : silu_mul(gate, up)) * so;
                } else {
                    if (g.bias) v += static_cast<const float *>(g.bias)[n];
                    if (g.epi == EPI_STREAMS) {
                        streams_column<float>(p.st, row, g.n, n, v);
                        continue;
                    }
                    if (g.epi == EPI_ADD_F32) v += *out;
                    if (g.epi == EPI_SOFTCAP_F32) v = g.limit * tanhf(v / g.limit);
                }
                *out = v;
            }
        }
    }
}

// Tiles the launch can have at most: families of experts share `rows` rows in an unknown way.
long tile_bound(const GemmParams &p, int bm, int bn_single, int bn_pair, const int *family_rows) {
    long t = 0;
    for (int g = 0; g < p.n_groups; g++) {
        const int bn = p.g[g].epi >= EPI_CLAMPED_GLU ? bn_pair : bn_single;
        const long nt = (p.g[g].n + bn - 1) / bn;
        if (p.g[g].experts > 0) {
            const long rows = family_rows[g];
            const long used = rows < p.g[g].experts ? rows : p.g[g].experts;
            t += nt * (used + rows / bm);
        } else {
            t += nt * ((p.g[g].rows + bm - 1) / bm);
        }
    }
    return t;
}

}  // namespace

int32_t encode_map(CUtensorMap *map, const void *base, int64_t rows, int64_t cols, int64_t pitch, int box_rows) {
    static PFN_cuTensorMapEncodeTiled_v12000 encode = [] {
        void *fn = nullptr;
        cudaDriverEntryPointQueryResult qres;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres) != cudaSuccess ||
            qres != cudaDriverEntryPointSuccess)
            fn = nullptr;
        cudaGetLastError();
        return reinterpret_cast<PFN_cuTensorMapEncodeTiled_v12000>(fn);
    }();
    TLC_REQUIRE(encode, TLC_ERR_DEVICE, "the driver has no cuTensorMapEncodeTiled");
    TLC_REQUIRE(((uintptr_t)base & 15) == 0 && (pitch & 7) == 0, TLC_ERR_INVALID_OPERATION,
                "tensor map: base and rows must be 16-byte aligned");
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)pitch * 2};
    const cuuint32_t box[2] = {(cuuint32_t)kBK, (cuuint32_t)box_rows};
    const cuuint32_t estr[2] = {1, 1};
    const CUresult rc = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, estr,
                               CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                               CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    TLC_REQUIRE(rc == CUDA_SUCCESS, TLC_ERR_CUDA, "tensor map of [%lld, %lld] refused (%d)", (long long)rows, (long long)cols, (int)rc);
    return TLC_OK;
}

static int32_t count_slots(GemmParams &p) {
    p.slots = 0;
    for (int g = 0; g < p.n_groups; g++) p.slots += p.g[g].experts > 0 ? p.g[g].experts : 1;
    TLC_REQUIRE(p.slots <= kMaxSlots, TLC_ERR_INVALID_OPERATION, "dense gemm: %d weights in one launch", p.slots);
    return TLC_OK;
}

template <int MAXS>
static int32_t launch_tensor(tlc_ctx *ctx, const GemmParams &p, long ctas) {
    static bool done[64] = {};
    constexpr size_t smem = kSmemD + (MAXS > 0 ? kSmemTurn : 0);
    if (!done[ctx->device & 63]) {
        TLC_CUDA(cudaFuncSetAttribute(dense_gemm_kernel<MAXS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        done[ctx->device & 63] = true;
    }
    cudaError_t le = tlc_launch_pdl(ctx, dense_gemm_kernel<MAXS>, dim3((unsigned)ctas), dim3(kThreadsD), smem, p);
    if (le != cudaSuccess) {
        cudaGetLastError();
        return tlc_fail(TLC_ERR_CUDA, "dense gemm launch failed: %s", cudaGetErrorString(le));
    }
    TLC_CHECK_LAUNCH(ctx);
    return TLC_OK;
}

template <>
int32_t launch_gemm<bf16>(tlc_ctx *ctx, GemmParams &p) {
    if (int32_t rc = count_slots(p)) return rc;
    p.status = ctx->dev_status;
    p.wait_ns = ctx->wait_ns;
    int family[6];
    for (int g = 0; g < p.n_groups; g++) family[g] = p.g[g].experts > 0 ? p.m * p.g[g].in_rows_per_token : 0;
    long tiles = tile_bound(p, 128, 256, 128, family);
    if (tiles > ctx->sm_count) tiles = ctx->sm_count;
    if (p.st.n == 0) return launch_tensor<0>(ctx, p, tiles);
    switch (p.st.n) {
        case 1: return launch_tensor<1>(ctx, p, tiles);
        case 2: return launch_tensor<2>(ctx, p, tiles);
        case 3: return launch_tensor<3>(ctx, p, tiles);
        case 4: return launch_tensor<4>(ctx, p, tiles);
        default: return launch_tensor<kMaxStreams>(ctx, p, tiles);
    }
}

template <>
int32_t launch_gemm<float>(tlc_ctx *ctx, GemmParams &p) {
    if (int32_t rc = count_slots(p)) return rc;
    p.status = ctx->dev_status;
    p.wait_ns = ctx->wait_ns;
    int family[6];
    for (int g = 0; g < p.n_groups; g++) family[g] = p.g[g].experts > 0 ? p.m * p.g[g].in_rows_per_token : 0;
    long tiles = tile_bound(p, 64, 64, 64, family);
    if (tiles > 4 * ctx->sm_count) tiles = 4 * ctx->sm_count;
    cudaError_t le = tlc_launch_pdl(ctx, dense_gemm_f32_kernel, dim3((unsigned)tiles), dim3(256), 0, p);
    if (le != cudaSuccess) {
        cudaGetLastError();
        return tlc_fail(TLC_ERR_CUDA, "f32 gemm launch failed: %s", cudaGetErrorString(le));
    }
    TLC_CHECK_LAUNCH(ctx);
    return TLC_OK;
}

}  // namespace tlc_dense
