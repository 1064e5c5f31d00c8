// On-device sampling shared by the model runners: greedy argmax and temperature sampling over f16
// or f32 logits, fused with the step bookkeeping (the sampled token becomes the next input, the
// sequence position advances) and with the report to pinned host memory.
#pragma once

#include "tlc_internal.h"
#include "tlc_synth.cuh"

// Where a decode step that runs as one graph reports to the host without copy nodes:
// pinned host words the sampling kernel writes directly (status first, then the token).
struct HostReport {
    int *host_next;                      // [batch] pinned, or null
    tlc_dev_status *host_status;         // pinned mirror of the status word
    const tlc_dev_status *dev_status;
};

// Uniform draw in [0, 1) with 24 bits, a pure function of (seed, position, sequence).
__host__ __device__ inline float tlc_sample_uniform(uint64_t seed, uint32_t pos, uint32_t seq) {
    const uint64_t r = tlc_mix64(tlc_mix64(seed ^ 0x73616d706c65ull) + ((uint64_t)pos << 20) + seq);
    return (float)(r >> 40) * (1.0f / 16777216.0f);
}

namespace tlc_sample {

__device__ __forceinline__ float logit_value(__half v) { return __half2float(v); }
__device__ __forceinline__ float logit_value(float v) { return v; }

__device__ __forceinline__ void report_to_host(const HostReport &hr, int b, int tok) {
    if (!hr.host_next) return;
    if (b == 0 && hr.host_status) {
        hr.host_status->code = hr.dev_status->code;
        hr.host_status->where = hr.dev_status->where;
    }
    __threadfence_system();
    *reinterpret_cast<volatile int *>(hr.host_next + b) = tok;
}

// Greedy sample + step bookkeeping, one CTA per sequence.  Ties go to the LAST
// maximal index, like Iterator::max_by in temperature_sample's greedy arm
// (src/interpreter/builtin_sampling.rs:176-181).  Also feeds the sampled token
// back as the next input and advances the sequence position.
// With tensor parallelism the logits arrive as gathered vocabulary shards
// [shard][row][vocab_per_shard]; token index = shard * vocab_per_shard + i.
template <typename LT>
__global__ void argmax_advance_kernel(const LT *__restrict__ logits, int vocab, int shards, int rows,
                                      int *__restrict__ next_ids, int *__restrict__ ids,
                                      int *__restrict__ positions, int advance, HostReport hr) {
    constexpr int VEC = 16 / (int)sizeof(LT);
    __shared__ float sv[32];
    __shared__ int si[32];
    tlc_pdl_prologue();  // the logits come from the previous kernel
    const int b = blockIdx.x;
    float best = -INFINITY;
    int bi = -1;
    for (int sh = 0; sh < shards; sh++) {
        const LT *row = logits + ((size_t)sh * rows + b) * vocab;
        if (vocab % VEC == 0 && (reinterpret_cast<uintptr_t>(row) & 15) == 0) {
            // 16-byte loads; a thread still meets its elements in increasing index order
            for (int c = threadIdx.x; c < vocab / VEC; c += blockDim.x) {
                const uint4 raw = *reinterpret_cast<const uint4 *>(row + VEC * c);
                const LT *h = reinterpret_cast<const LT *>(&raw);
#pragma unroll
                for (int j = 0; j < VEC; j++) {
                    const float v = logit_value(h[j]);
                    if (bi < 0 || !(v < best)) {
                        best = v;
                        bi = sh * vocab + VEC * c + j;
                    }
                }
            }
            continue;
        }
        for (int i = threadIdx.x; i < vocab; i += blockDim.x) {
            const float v = logit_value(row[i]);
            if (bi < 0 || !(v < best)) {  // v >= best (or unordered): later index wins
                best = v;
                bi = sh * vocab + i;
            }
        }
    }
    auto better = [](float v, int i, float bv, int bidx) {
        if (bidx < 0) return true;
        if (i < 0) return false;
        if (v > bv) return true;
        if (v < bv) return false;
        return i > bidx;
    };
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (better(ov, oi, best, bi)) {
            best = ov;
            bi = oi;
        }
    }
    if ((threadIdx.x & 31) == 0) {
        sv[threadIdx.x >> 5] = best;
        si[threadIdx.x >> 5] = bi;
    }
    __syncthreads();
    if (threadIdx.x < 32) {
        const int nw = blockDim.x >> 5;
        best = threadIdx.x < nw ? sv[threadIdx.x] : -INFINITY;
        bi = threadIdx.x < nw ? si[threadIdx.x] : -1;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (better(ov, oi, best, bi)) {
                best = ov;
                bi = oi;
            }
        }
        if (threadIdx.x == 0) {
            next_ids[b] = bi;
            if (advance) {
                ids[b] = bi;
                positions[b] += 1;
            }
            report_to_host(hr, b, bi);
        }
    }
}

// Temperature sample + step bookkeeping, one CTA per sequence: the arithmetic of
// temperature_sample_cpu (src/interpreter/builtin_sampling.rs:185-217) -- logits
// widened to f32 and divided by the temperature, softmax with the maximum
// subtracted, first index whose running probability sum exceeds the uniform
// draw, the last index if none does -- with the sums formed in parallel: every
// thread owns a contiguous run of the vocabulary, a block-wide scan gives each
// run its starting sum, and the comparison is made against u * total instead of
// dividing every probability (the f32 rounding differs from the sequential sum
// only for draws within ~1e-6 of a boundary).
// u comes from `uniforms[b]` when given, else from tlc_sample_uniform; row b belongs to sequence
// seq0 + b.
template <typename LT>
__global__ void __launch_bounds__(1024) sample_advance_kernel(const LT *__restrict__ logits, int vocab, int shards,
                                                              int rows, float temperature, uint64_t seed,
                                                              const float *__restrict__ uniforms, int fixed_pos, int seq0,
                                                              int *__restrict__ next_ids, int *__restrict__ ids,
                                                              int *__restrict__ positions, int advance, HostReport hr) {
    __shared__ float red[32];
    __shared__ float warp_sum[32];
    __shared__ int found_min;
    tlc_pdl_prologue();  // the logits come from the previous kernel
    const int b = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int V = vocab * shards;
    const int seg = (V + (int)blockDim.x - 1) / (int)blockDim.x;
    const int lo = min(V, tid * seg), hi = min(V, lo + seg);
    auto logit = [&](int j) {  // token j of the gathered shards
        const int sh = j / vocab, i = j - sh * vocab;
        return logit_value(logits[((size_t)sh * rows + b) * vocab + i]) / temperature;
    };
    float mx = -INFINITY;
    for (int j = lo; j < hi; j++) mx = fmaxf(mx, logit(j));
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    if (lane == 0) red[warp] = mx;
    if (tid == 0) found_min = V - 1;  // "default to last token"
    __syncthreads();
    mx = red[lane];  // blockDim.x == 1024: 32 warps
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float local = 0.f;
    for (int j = lo; j < hi; j++) local += expf(logit(j) - mx);
    // inclusive scan of the per-thread sums: within the warp, then across warps
    float incl = local;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float t = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += t;
    }
    if (lane == 31) warp_sum[warp] = incl;
    __syncthreads();
    float wbase = 0.f, total = 0.f;
    {
        float w = warp_sum[lane], wi = w;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float t = __shfl_up_sync(0xffffffffu, wi, o);
            if (lane >= o) wi += t;
        }
        total = __shfl_sync(0xffffffffu, wi, 31);
        wbase = __shfl_sync(0xffffffffu, wi - w, warp);  // exclusive sum of the warps before this one
    }
    const int pos = fixed_pos >= 0 ? fixed_pos : positions ? positions[b] : 0;  // position of the token fed to this step
    const float u = uniforms ? uniforms[b] : tlc_sample_uniform(seed, (uint32_t)pos, (uint32_t)(seq0 + b));
    const float target = u * total;
    float run = wbase + incl - local;  // sum of everything before this thread's run
    if (target < run + local) {
        for (int j = lo; j < hi; j++) {
            run += expf(logit(j) - mx);
            if (target < run) {
                atomicMin(&found_min, j);
                break;
            }
        }
    }
    __syncthreads();
    if (tid == 0) {
        const int tok = found_min;
        next_ids[b] = tok;
        if (advance) {
            ids[b] = tok;
            positions[b] += 1;
        }
        report_to_host(hr, b, tok);
    }
}

}  // namespace tlc_sample
