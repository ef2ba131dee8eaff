// Shared by the kernels of the layer-list ("hybrid") models: element types, block reductions,
// the row index of a position in a key/value cache, and the set of keys a query sees.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../../include/mkb200_hybrid.h"
#include "mk_common.cuh"

namespace mkbh {

using bf16 = __nv_bfloat16;

constexpr int kMaxRowBytes = 32768;  // longest row of a weight matrix (checked on the host)

__host__ __device__ inline int pad8(int n) { return (n + 7) & ~7; }

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum of N values per thread over a block of kThreads; every thread gets the totals.
// `red` holds N * (kThreads / 32) floats and may be reused after the next block barrier.
template <int N, int kThreads>
__device__ __forceinline__ void block_sum(float (&v)[N], float* red) {
    constexpr int W = kThreads / 32;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
    for (int n = 0; n < N; ++n) {
        v[n] = warp_sum(v[n]);
        if (lane == 0) red[n * W + warp] = v[n];
    }
    __syncthreads();
#pragma unroll
    for (int n = 0; n < N; ++n) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < W; ++w) s += red[n * W + w];
        v[n] = s;
    }
    __syncthreads();
}

// Row of position j in a cache that keeps the first `keep` positions for good and the later
// ones in a ring.
__host__ __device__ inline int cache_row(int j, int keep, int ring) {
    return j < keep ? j : keep + (j - keep) % ring;
}

// Keys that the query at `pos` sees: the first `sinks` positions, then `count - sinks` positions
// from `start` on, up to the query itself: its window, or its chunk (chunks count from position 0).
struct KeyRange {
    int sinks, start, count;
    __host__ __device__ KeyRange(int pos, int window, int keep_first, int chunk) {
        const int n = chunk > 0 ? pos % chunk + 1 : pos + 1 < window ? pos + 1 : window;
        start = pos + 1 - n;
        sinks = chunk > 0 ? 0 : keep_first < start ? keep_first : start;
        count = sinks + n;
    }
    __host__ __device__ int key(int t) const { return t < sinks ? t : start + (t - sinks); }
};

// Sizes of a layer's mixer.
__host__ __device__ inline bool is_attention(const MkbhLayer& L) { return L.mixer != MKBH_DELTA_RULE; }
__host__ __device__ inline int mixer_out(const MkbhLayer& L) { return L.heads * (L.mixer == MKBH_DELTA_RULE ? L.dim : L.vdim); }
__host__ __device__ inline int latent_dim(const MkbhLayer& L) { return pad8(L.rank) + pad8(L.rot_dim); }
// Elements from one latent to the next: an odd number of eights (rows that start in different banks).
__host__ __device__ inline int latent_row(const MkbhLayer& L) { return (latent_dim(L) / 8 | 1) * 8; }
__host__ __device__ inline int up_rows(const MkbhLayer& L) { return L.ff_kind == MKBH_CLAMPED_GLU ? 2 * L.ff : L.ff; }
// Phase whose end makes the mixer's output complete.
__host__ __device__ inline int mixer_phase(int mixer) {
    return mixer == MKBH_DELTA_RULE ? MKBH_OP_DELTA_STEP : mixer == MKBH_LATENT_ATTENTION ? MKBH_OP_EXPAND : MKBH_OP_ATTENTION;
}

// Gated unit with clamped halves: g' sigmoid(alpha g') (u' + 1).
__device__ __forceinline__ float clamped_glu(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoid_f(alpha * g) * (u + 1.f);
}

}  // namespace mkbh
