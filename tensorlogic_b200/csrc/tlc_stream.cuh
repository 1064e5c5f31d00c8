// Streaming weight rows against one input: the pieces the one-row kernels share.
#pragma once

#include "tlc_dense.cuh"

#ifdef __CUDACC__
namespace tlc_dense {

constexpr int kBatch = 4;  // 16-byte loads of a lane per batch; two batches are in flight

// Input layout in shared memory: piece c (16 bytes of weights) faces floats 4 c .. 4 c + 3 of plane
// 0 and, for bf16, of plane 1, so that a warp's 16-byte reads fall on distinct banks.

// Piece c of an input of `pieces`, as f32 in its places.
template <typename T>
__device__ __forceinline__ void put_piece(float *in, int c, int pieces, const float (&f)[Vec<T>::N]) {
    *reinterpret_cast<float4 *>(in + 4 * c) = make_float4(f[0], f[1], f[2], f[3]);
    if constexpr (Vec<T>::N == 8) *reinterpret_cast<float4 *>(in + 4 * (pieces + c)) = make_float4(f[4], f[5], f[6], f[7]);
}
template <typename T>
__device__ __forceinline__ void get_piece(const float *in, int c, int pieces, float (&f)[Vec<T>::N]) {
    const float4 a = *reinterpret_cast<const float4 *>(in + 4 * c);
    f[0] = a.x;
    f[1] = a.y;
    f[2] = a.z;
    f[3] = a.w;
    if constexpr (Vec<T>::N == 8) {
        const float4 b = *reinterpret_cast<const float4 *>(in + 4 * (pieces + c));
        f[4] = b.x;
        f[5] = b.y;
        f[6] = b.z;
        f[7] = b.w;
    }
}
// Piece c of n f32 values (rows start on 16-byte boundaries), zeros past n.
template <typename T>
__device__ __forceinline__ void load_f32_piece(const float *x, int c, int n, float (&f)[Vec<T>::N]) {
    constexpr int N = Vec<T>::N;
    if (N * c + N <= n) {
#pragma unroll
        for (int j = 0; j < N; j += 4) {
            const float4 v = __ldcg(reinterpret_cast<const float4 *>(x + N * c + j));
            f[j] = v.x;
            f[j + 1] = v.y;
            f[j + 2] = v.z;
            f[j + 3] = v.w;
        }
    } else {
#pragma unroll
        for (int j = 0; j < N; j++) f[j] = N * c + j < n ? __ldcg(x + N * c + j) : 0.f;
    }
}
// Zeroes the values of piece c from n on.
template <typename T>
__device__ __forceinline__ void cut_piece(int c, int n, float (&f)[Vec<T>::N]) {
#pragma unroll
    for (int j = 0; j < Vec<T>::N; j++)
        if (Vec<T>::N * c + j >= n) f[j] = 0.f;
}

__device__ __forceinline__ uint4 load_weight(const uint4 *p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];"
                 : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
                 : "l"(p));
    return v;
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

// A stretch of one weight row: pieces [lo, hi) of w against the input pieces of the same numbers
// plus `shift`; its sum times `scale` goes to part[slot].
struct Item {
    const uint4 *w;
    int lo, hi, shift, slot;
    float scale;
};

// The items of a CTA of WARPS warps: `rows` rows of `per_row` stretches each; warp w takes items w, w + WARPS, ...
// in row order.  `item(row, stretch)` describes one.
template <typename T, int WARPS, typename F>
__device__ __forceinline__ void stream_items(int rows, int per_row, const float *plane0, const float *plane1, float *part, F item) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int dr = WARPS / per_row, dt = WARPS - dr * per_row;
    struct Cursor {
        int r, t;
        Item it;
    };
    auto advance = [&](Cursor &c) {
        c.r += dr;
        c.t += dt;
        if (c.t >= per_row) {
            c.t -= per_row;
            c.r++;
        }
        if (c.r < rows) c.it = item(c.r, c.t);
    };
    Cursor ld;
    ld.r = warp / per_row;
    ld.t = warp - ld.r * per_row;
    if (ld.r >= rows) return;
    ld.it = item(ld.r, ld.t);
    Cursor use = ld;
    float acc = 0.f;
    auto load_batch = [&](uint4 (&w)[kBatch]) {
        if (ld.r >= rows) return;
        const uint4 *src = ld.it.w + ld.it.lo + lane;
        const int left = ld.it.hi - ld.it.lo - lane;
#pragma unroll
        for (int u = 0; u < kBatch; u++)
            if (32 * u < left) w[u] = load_weight(src + 32 * u);
        ld.it.lo += 32 * kBatch;
        if (ld.it.lo >= ld.it.hi) advance(ld);
    };
    auto use_batch = [&](uint4 (&w)[kBatch]) {
        const int c = use.it.lo + lane, left = use.it.hi - c;
#pragma unroll
        for (int u = 0; u < kBatch; u++)
            if (32 * u < left) acc += dot_piece<T>(w[u], plane0, plane1, c + 32 * u + use.it.shift);
        use.it.lo += 32 * kBatch;
        if (use.it.lo >= use.it.hi) {
            acc = warp_sum(acc);
            if (lane == 0) part[use.it.slot] = acc * use.it.scale;
            acc = 0.f;
            advance(use);
        }
    };
    uint4 a[kBatch], b[kBatch];
    load_batch(a);
    while (use.r < rows) {
        load_batch(b);
        use_batch(a);
        if (use.r >= rows) break;
        load_batch(a);
        use_batch(b);
    }
}

// Stretch `part` of a row of `pieces` cut every `per` pieces.
__device__ __forceinline__ void share_of(int per, int pieces, int part, Item &it) {
    const int lo = part * per;
    it.lo = lo < pieces ? lo : pieces;
    it.hi = lo + per < pieces ? lo + per : pieces;
}

}  // namespace tlc_dense
#endif
