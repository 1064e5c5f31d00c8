// Latent attention, expanded form: consecutive rows of one sequence against keys and values made from the
// cache's latents for the whole stretch (bf16, tcgen05).
//
// One CTA takes 128 queries of one head.  Keys come in tiles of 64: unrotated parts from k_all, the
// rotated part all heads share straight from the cache, values transposed (V rows of 64 keys), so that
// every operand is K-major; all by TMA with the 128-byte swizzle, two to four stages.
//   warp 0       TMA
//   warp 1       issues S = Q K^T, as far ahead as there are score buffers (four; two when the accumulators
//                leave no more room in the tensor memory)
//   warp 2       issues P V
//   warps 3-10   two softmax groups of 128 threads, one query row per thread; group g owns the tiles
//                j = g (mod 2), its own accumulator, maximum and sum, so the groups never wait for one
//                another before the end.  The weights P take the place of the scores in tensor memory.
// Issuing an MMA takes about as long as running one of this size: hence two issuing warps, each of
// which runs its loop as a whole (descriptors in uniform registers) and elects the issuing thread.
// A group's accumulator is rescaled only when a row's maximum has grown by more than 2^8; weights are
// relative to the maximum of the last rescaling, so they stay below 2^8.  A weight enters the P.V product
// as the sum of two bf16 numbers.  At the end the two accumulators and the sink are merged.
// All waits are bounded; a wait that runs out sets the status word and lets the CTA drain, free its tensor
// memory and return.
#include "tlc_dense.cuh"
#include "tlc_gemm_kernel.cuh"
#include "tlc_mma.cuh"

namespace tlc_dense {

namespace {

using tlc_gemm::fence_async_proxy;
using tlc_gemm::make_desc;
using tlc_gemm::mbar_arrive;
using tlc_gemm::mbar_arrive_expect_tx;
using tlc_gemm::mbar_init;
using tlc_gemm::mbar_wait;
using tlc_gemm::smem_u32;
using tlc_gemm::tc_fence_after;
using tlc_gemm::tc_fence_before;
using tlc_gemm::tma_load_2d;
using tlc_gemm::tmem_ld32;
using tlc_gemm::umma_commit;
using tlc_gemm::umma_f16;

constexpr int kRows = 128, kTile = 64;
constexpr int kGroup = 128, kThreadsP = 96 + 2 * kGroup;
constexpr int kQChunk = kRows * 128, kKChunk = kTile * 128;  // bytes of 64 columns
constexpr int kMaxStages = 4;
constexpr uint32_t kIdesc = (1u << 7) | (1u << 10);          // bf16 x bf16
constexpr float kLog2e = 1.44269504088896340736f;
constexpr size_t kSmemLimit = 226 * 1024, kExtra = 256 + 4 * kRows * sizeof(float);

struct Layout {  // of the shared memory, in bytes from a 1024-byte boundary
    int chunks_d, chunks_r, v_rows, stages;
    size_t k_stage, v_stage, k, v, bars, total;
    __host__ __device__ Layout(int D, int R, int V)
        : chunks_d((D + 63) / 64), chunks_r((R + 63) / 64), v_rows((V + 63) / 64 * 64), k_stage((size_t)(chunks_d + chunks_r) * kKChunk),
          v_stage((size_t)v_rows * 128), k((size_t)(chunks_d + chunks_r) * kQChunk) {
        const size_t room = kSmemLimit > k + kExtra ? kSmemLimit - k - kExtra : 0;
        stages = (int)(room / (k_stage + v_stage));
        if (stages > kMaxStages) stages = kMaxStages;
        v = k + stages * k_stage;
        bars = v + stages * v_stage;
        total = bars + kExtra;
    }
};

struct Bars {
    uint64_t q_full, q_ready, k_full[kMaxStages], k_empty[kMaxStages], v_full[kMaxStages], v_empty[kMaxStages], s_full[4], p_full[4], o_done[4];
    uint32_t tmem;
    int abort;
};
struct Ring {  // position in a ring of stages
    int at = 0;
    uint32_t parity = 0;
    __device__ __forceinline__ void next(int stages) {
        if (++at == stages) {
            at = 0;
            parity ^= 1u;
        }
    }
};

// A wait in the chain from one tile to the next: polls first, then the timed wait.
__device__ __forceinline__ bool wait_soon(uint64_t *bar, uint32_t parity, volatile int *abort_flag, tlc_dev_status *status, int where,
                                          uint64_t wait_ns) {
    for (int i = 0; i < 64; i++)
        if (tlc_gemm::mbar_try_wait(bar, parity)) return true;
    return mbar_wait(bar, parity, abort_flag, status, where, wait_ns);
}
// One thread of the warp.
__device__ __forceinline__ bool elect_one() {
    uint32_t p;
    asm volatile("{\n .reg .pred q;\n elect.sync _|q, 0xffffffff;\n selp.u32 %0, 1, 0, q;\n}\n" : "=r"(p));
    return p != 0;
}
// 2^x; results below the normal numbers are zero.
__device__ __forceinline__ float exp2_ftz(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t (&r)[16]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
          "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(taddr));
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%16], {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15};" ::"r"(r[0]), "r"(r[1]),
        "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]),
        "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(taddr)
        : "memory");
    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
}

__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t (&r)[32]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%32], "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,"
        "%29,%30,%31};" ::"r"(r[0]),
        "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]),
        "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]),
        "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31]), "r"(taddr)
        : "memory");
}
// D += A B with A (bf16, two values per 32-bit column, a row per lane) in tensor memory.
__device__ __forceinline__ void umma_f16_tmem_a(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
        " tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n}\n" ::"r"(tmem_d),
        "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}

__global__ void __launch_bounds__(kThreadsP, 1) latent_prefill_kernel(const __grid_constant__ LatentParams p) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *base = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const Layout lay(p.D, p.R, p.V);
    Bars *b = reinterpret_cast<Bars *>(base + lay.bars);
    float *stat = reinterpret_cast<float *>(base + lay.bars + 256);  // [2][128] maxima, [2][128] sums
    volatile int *abort_flag = &b->abort;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int head = blockIdx.x, row0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * kRows;  // later rows first: they have the most keys
    const int last_row = row0 + kRows < p.m ? row0 + kRows - 1 : p.m - 1;
    const int n_tiles = (p.pos0 + last_row) / kTile + 1;
    if (tid == 0) {
        mbar_init(&b->q_full, 1);
        mbar_init(&b->q_ready, 2 * kGroup);
        for (int s = 0; s < kMaxStages; s++) {
            mbar_init(&b->k_full[s], 1);
            mbar_init(&b->k_empty[s], 1);
            mbar_init(&b->v_full[s], 1);
            mbar_init(&b->v_empty[s], 1);
        }
        for (int s = 0; s < 4; s++) {
            mbar_init(&b->s_full[s], 1);
            mbar_init(&b->p_full[s], kGroup);
            mbar_init(&b->o_done[s], 1);
        }
        b->abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&b->tmem)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = b->tmem;
    const int ahead = 4 * kTile + 2 * p.V <= 512 ? 4 : 2;  // score buffers
    const uint32_t tm_o[2] = {tmem + ahead * kTile, tmem + ahead * kTile + (uint32_t)p.V};
    pdl_enter();

    if (warp == 0) {
        if (lane == 0) {
            const int x_q = head * (p.D + p.R), x_k = head * p.D;
            {
                mbar_arrive_expect_tx(&b->q_full, (uint32_t)((lay.chunks_d + lay.chunks_r) * kQChunk));
                const uint32_t at = smem_u32(base), bar = smem_u32(&b->q_full);
                for (int c = 0; c < lay.chunks_d; c++) tma_load_2d(at + c * kQChunk, p.q_map, x_q + 64 * c, row0, bar);
                for (int c = 0; c < lay.chunks_r; c++)
                    tma_load_2d(at + (lay.chunks_d + c) * kQChunk, p.q_map, x_q + p.D + 64 * c, row0, bar);
            }
            int nk = 0, nv = 0;  // tiles asked for
            Ring rk, rv;
            auto load_k = [&] {
                if (!mbar_wait(&b->k_empty[rk.at], rk.parity ^ 1u, abort_flag, p.status, 31, p.wait_ns)) return false;
                mbar_arrive_expect_tx(&b->k_full[rk.at], (uint32_t)lay.k_stage);
                const uint32_t at = smem_u32(base + lay.k + rk.at * lay.k_stage), bar = smem_u32(&b->k_full[rk.at]);
                for (int c = 0; c < lay.chunks_d; c++) tma_load_2d(at + c * kKChunk, p.k_map, x_k + 64 * c, nk * kTile, bar);
                for (int c = 0; c < lay.chunks_r; c++)
                    tma_load_2d(at + (lay.chunks_d + c) * kKChunk, p.rot_map, 64 * c, p.slot0 * p.max_seq + nk * kTile, bar);
                nk++;
                rk.next(lay.stages);
                return true;
            };
            auto load_v = [&] {
                if (!mbar_wait(&b->v_empty[rv.at], rv.parity ^ 1u, abort_flag, p.status, 32, p.wait_ns)) return false;
                mbar_arrive_expect_tx(&b->v_full[rv.at], (uint32_t)lay.v_stage);
                const uint32_t at = smem_u32(base + lay.v + rv.at * lay.v_stage), bar = smem_u32(&b->v_full[rv.at]);
                for (int r = 0; r < lay.v_rows; r += 64) tma_load_2d(at + r * 128, p.v_map, nv * kTile, head * p.V + r, bar);
                nv++;
                rv.next(lay.stages);
                return true;
            };
            // keys two tiles ahead of the values, as their products
            bool ok = load_k() && (n_tiles < 2 || load_k());
            while (ok && nv < n_tiles) ok = load_v() && (nk == n_tiles || load_k());
            if (*abort_flag) {  // no copy may be in flight when the CTA ends: the last ones of every stage
                mbar_wait(&b->q_full, 0, abort_flag, p.status, 33, p.wait_ns);
                for (int i = nk > lay.stages ? nk - lay.stages : 0; i < nk; i++)
                    mbar_wait(&b->k_full[i % lay.stages], (i / lay.stages) & 1u, abort_flag, p.status, 33, p.wait_ns);
                for (int i = nv > lay.stages ? nv - lay.stages : 0; i < nv; i++)
                    mbar_wait(&b->v_full[i % lay.stages], (i / lay.stages) & 1u, abort_flag, p.status, 33, p.wait_ns);
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        const uint32_t idesc = tlc_gemm::idesc_for(kTile) | kIdesc;
        const uint64_t qd = make_desc(smem_u32(base)), kd = make_desc(smem_u32(base + lay.k));
        const uint32_t step = (uint32_t)(lay.k_stage >> 4);  // descriptors count 16 bytes
        const int chunks = lay.chunks_d + lay.chunks_r;
        Ring ring, bufs;
        bool ok = mbar_wait(&b->q_ready, 0, abort_flag, p.status, 35, p.wait_ns);
        for (int j = 0; j < n_tiles; j++) {
            // the buffer held the weights of tile j - ahead: their product must be complete
            if (j >= ahead) ok = ok && wait_soon(&b->o_done[bufs.at], bufs.parity ^ 1u, abort_flag, p.status, 42, p.wait_ns);
            ok = ok && wait_soon(&b->k_full[ring.at], ring.parity, abort_flag, p.status, 34, p.wait_ns);
            if (!__all_sync(0xffffffffu, ok)) break;
            tc_fence_after();
            const uint32_t to = tmem + bufs.at * kTile;
            const uint64_t ks = kd + ring.at * step;
            if (elect_one()) {
                for (int c = 0; c < chunks; c++) {  // 64 columns: four steps of 16, fewer at the end of a part
                    const int steps = c < lay.chunks_d ? p.D / 16 - 4 * c : p.R / 16 - 4 * (c - lay.chunks_d);
                    const uint64_t qc = qd + c * (kQChunk >> 4), kc = ks + c * (kKChunk >> 4);
                    umma_f16(to, qc, kc, idesc, c > 0 ? 1u : 0u);
#pragma unroll
                    for (int kk = 1; kk < 4; kk++)
                        if (kk < steps) umma_f16(to, qc + 2 * kk, kc + 2 * kk, idesc, 1u);
                }
                umma_commit(&b->k_empty[ring.at]);
                umma_commit(&b->s_full[bufs.at]);
            }
            __syncwarp();
            ring.next(lay.stages);
            bufs.next(ahead);
        }
    } else if (warp == 2) {
        const uint32_t idesc = tlc_gemm::idesc_for(p.V) | kIdesc;
        const uint64_t vd = make_desc(smem_u32(base + lay.v));
        const uint32_t step = (uint32_t)(lay.v_stage >> 4);
        Ring ring, bufs;
        for (int j = 0; j < n_tiles; j++) {
            const bool ok = wait_soon(&b->p_full[bufs.at], bufs.parity, abort_flag, p.status, 36, p.wait_ns) &&
                            wait_soon(&b->v_full[ring.at], ring.parity, abort_flag, p.status, 37, p.wait_ns);
            if (!__all_sync(0xffffffffu, ok)) break;
            tc_fence_after();
            const uint32_t pa = tmem + bufs.at * kTile, to = tmem + ahead * kTile + (j & 1) * p.V;
            const uint64_t vs = vd + ring.at * step;
            if (elect_one()) {
                umma_f16_tmem_a(to, pa, vs, idesc, j > 1 ? 1u : 0u);
#pragma unroll
                for (int i = 1; i < kTile / 8; i++)  // the high parts of the weights, then the low ones
                    umma_f16_tmem_a(to, pa + 8 * i, vs + 2 * (i & 3), idesc, 1u);
                umma_commit(&b->v_empty[ring.at]);
                umma_commit(&b->o_done[bufs.at]);
            }
            __syncwarp();
            ring.next(lay.stages);
            bufs.next(ahead);
        }
    } else {
        const int g = (warp - 3) >> 2, wq = warp & 3, r = 32 * wq + lane;  // tensor-memory lanes this warp may touch: 32 wq ..
        const uint32_t lanes = (uint32_t)(32 * wq) << 16;
        const int pos = p.pos0 + row0 + r, warp_first = p.pos0 + row0 + 32 * wq;
        // rotate the queries: the groups share a row's pairs
        mbar_wait(&b->q_full, 0, abort_flag, p.status, 38, p.wait_ns);
        for (int i = 4 * g; i < p.R / 2; i += 8) {  // four pairs: one 16-byte piece
            const int e = 2 * i, c = e >> 6, piece = (e & 63) >> 3;
            uint4 *at = reinterpret_cast<uint4 *>(base + (size_t)(lay.chunks_d + c) * kQChunk + r * 128 + ((piece ^ (r & 7)) << 4));
            float f[8];
            unpack(*at, f);
            uint32_t o[4];
#pragma unroll
            for (int t = 0; t < 4; t++) {
                float sn, cs;
                sincosf((float)pos * __ldg(p.freq + i + t), &sn, &cs);
                o[t] = pack_bf16(f[2 * t] * cs - f[2 * t + 1] * sn, f[2 * t + 1] * cs + f[2 * t] * sn);
            }
            *at = make_uint4(o[0], o[1], o[2], o[3]);
        }
        fence_async_proxy();
        mbar_arrive(&b->q_ready);

        const float scale2 = p.scale * kLog2e;
        float m = -INFINITY, l = 0.f;
        // buffer and phase of a tile
        auto buffer = [&](int j) { return j & (ahead - 1); };
        auto phase = [&](int j) { return (uint32_t)(ahead == 4 ? j >> 2 : j >> 1) & 1u; };
        int it = 0;
        for (int j = g; j < n_tiles; j += 2, it++) {
            const int buf = buffer(j);
            wait_soon(&b->s_full[buf], phase(j), abort_flag, p.status, 39, p.wait_ns);
            tc_fence_after();
            uint32_t s[2][32];
            tmem_ld32(tmem + buf * kTile + lanes, s[0]);
            tmem_ld32(tmem + buf * kTile + lanes + 32, s[1]);
            const int j0 = j * kTile;
            float mx0 = -INFINITY, mx1 = -INFINITY;
            if (j0 + kTile - 1 > warp_first) {  // some row of the warp does not see every key
#pragma unroll
                for (int e = 0; e < 32; e++) {
                    if (j0 + e > pos) s[0][e] = 0xff800000u;
                    if (j0 + 32 + e > pos) s[1][e] = 0xff800000u;
                }
            }
#pragma unroll
            for (int e = 0; e < 32; e++) {
                mx0 = fmaxf(mx0, __uint_as_float(s[0][e]));
                mx1 = fmaxf(mx1, __uint_as_float(s[1][e]));
            }
            const float top = fmaxf(mx0, mx1) * scale2;  // the scale is positive
            if (it == 0) {
                m = top;
            } else if (__any_sync(0xffffffffu, top > m + 8.f)) {
                wait_soon(&b->o_done[buffer(j - 2)], phase(j - 2), abort_flag, p.status, 40, p.wait_ns);
                const float m_new = fmaxf(m, top), f = m_new == -INFINITY ? 1.f : exp2f(m - m_new);
                tc_fence_after();
#pragma unroll 1
                for (int c = 0; c < p.V; c += 16) {
                    uint32_t o[16];
                    tmem_ld16(tm_o[g] + lanes + c, o);
#pragma unroll
                    for (int e = 0; e < 16; e++) o[e] = __float_as_uint(__uint_as_float(o[e]) * f);
                    tmem_st16(tm_o[g] + lanes + c, o);
                }
                l *= f;
                m = m_new;
            }
            const float from = m == -INFINITY ? 0.f : m;
            float sum0 = 0.f, sum1 = 0.f;
            uint32_t hi[32], lo[32];
#pragma unroll
            for (int c = 0; c < 2; c++) {
#pragma unroll
                for (int e = 0; e < 32; e += 2) {
                    const float a = exp2_ftz(fmaf(__uint_as_float(s[c][e]), scale2, -from));
                    const float d = exp2_ftz(fmaf(__uint_as_float(s[c][e + 1]), scale2, -from));
                    sum0 += a;
                    sum1 += d;
                    split_pair(a, d, hi[16 * c + e / 2], lo[16 * c + e / 2]);
                }
            }
            tmem_st32(tmem + buf * kTile + lanes, hi);
            tmem_st32(tmem + buf * kTile + lanes + kTile / 2, lo);
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            l += sum0 + sum1;
            tc_fence_before();
            mbar_arrive(&b->p_full[buf]);
        }
        if (it > 0) {
            const int last = g + 2 * (it - 1);
            mbar_wait(&b->o_done[buffer(last)], phase(last), abort_flag, p.status, 41, p.wait_ns);
        }
        stat[g * kRows + r] = m;
        stat[(2 + g) * kRows + r] = l;
        tc_fence_before();
        asm volatile("bar.sync 1, 256;" ::: "memory");
        tc_fence_after();
        const float sink = to_f32(static_cast<const bf16 *>(p.sink)[head]) * kLog2e;
        const float m0 = stat[r], m1 = stat[kRows + r], top = fmaxf(fmaxf(m0, m1), sink);
        const float e0 = exp2f(m0 - top), e1 = exp2f(m1 - top);
        const float inv = 1.f / (stat[2 * kRows + r] * e0 + stat[3 * kRows + r] * e1 + exp2f(sink - top));
        const float f0 = e0 * inv, f1 = e1 * inv;
        const bool two = n_tiles > 1;  // else the second accumulator was never written
        bf16 *out = static_cast<bf16 *>(p.out) + (size_t)(row0 + r) * p.ldo + (size_t)head * p.V;
        const bool store = row0 + r < p.m && !*abort_flag;
        for (int c = 16 * g; c < p.V; c += 32) {  // the groups take 16 columns in turn
            uint32_t a[16], d[16];
            tmem_ld16(tm_o[0] + lanes + c, a);
            tmem_ld16(tm_o[1] + lanes + c, d);
            uint32_t o[8];
#pragma unroll
            for (int t = 0; t < 8; t++) {
                float u = __uint_as_float(a[2 * t]) * f0, v = __uint_as_float(a[2 * t + 1]) * f0;
                if (two) {
                    u += __uint_as_float(d[2 * t]) * f1;
                    v += __uint_as_float(d[2 * t + 1]) * f1;
                }
                o[t] = pack_bf16(u, v);
            }
            if (store) {
                *reinterpret_cast<uint4 *>(out + c) = make_uint4(o[0], o[1], o[2], o[3]);
                *reinterpret_cast<uint4 *>(out + c + 8) = make_uint4(o[4], o[5], o[6], o[7]);
            }
        }
        tc_fence_before();
    }
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
    }
}

}  // namespace

bool latent_prefill_fits(int D, int R, int V, float scale) {
    static_assert(sizeof(Bars) <= 256, "the barriers have 256 bytes");
    return scale > 0.f && D % 16 == 0 && R % 16 == 0 && V % 16 == 0 && D > 0 && V > 0 && 2 * kTile + 2 * V <= 512 && D + R <= 512 &&
           Layout(D, R, V).stages >= 2;
}

int32_t launch_latent_prefill(tlc_ctx *ctx, const LatentParams &p) {
    TLC_REQUIRE(latent_prefill_fits(p.D, p.R, p.V, p.scale), TLC_ERR_INVALID_OPERATION, "latent attention: heads of %d + %d and %d values", p.D,
                p.R, p.V);
    static bool done[64] = {};
    if (!done[ctx->device & 63]) {
        TLC_CUDA(cudaFuncSetAttribute(latent_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        done[ctx->device & 63] = true;
    }
    cudaError_t le = tlc_launch_pdl(ctx, latent_prefill_kernel, dim3((unsigned)p.H, (unsigned)((p.m + kRows - 1) / kRows)), dim3(kThreadsP),
                                    Layout(p.D, p.R, p.V).total + 1024, p);
    if (le != cudaSuccess) {
        cudaGetLastError();
        return tlc_fail(TLC_ERR_CUDA, "latent attention launch failed: %s", cudaGetErrorString(le));
    }
    TLC_CHECK_LAUNCH(ctx);
    return TLC_OK;
}

}  // namespace tlc_dense
