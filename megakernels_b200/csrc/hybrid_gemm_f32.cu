// 32-bit matrix product of the hybrid models' float build (true fp32 FMA, no reduced-precision
// matrix mode): 64 x 64 tiles, 4 x 4 outputs per thread.
#include "hybrid_kernels.h"

namespace mkbh {
namespace {

constexpr int kTile = 64, kDepth = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, int64_t lda,
                                                       const float* __restrict__ W, int64_t ldw, int T, int N, int K,
                                                       GemmEpilogue e) {
    __shared__ float sa[kDepth][kTile + 4], sw[kDepth][kTile + 4];
    const int n0 = blockIdx.x * kTile, t0 = blockIdx.y * kTile, tid = threadIdx.x;
    const int tx = tid & 15, ty = tid >> 4;
    const int lr = tid >> 2, lc = (tid & 3) * 4;  // one float4 of each operand per thread and step
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += kDepth) {
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f), w = a;
        if (k0 + lc < K) {  // (rows are padded to 8: what lies beyond K may be read, and is dropped)
            if (t0 + lr < T) a = *reinterpret_cast<const float4*>(A + (size_t)(t0 + lr) * lda + k0 + lc);
            if (n0 + lr < N) w = *reinterpret_cast<const float4*>(W + (size_t)(n0 + lr) * ldw + k0 + lc);
            if (k0 + lc + 1 >= K) a.y = 0.f;
            if (k0 + lc + 2 >= K) a.z = 0.f;
            if (k0 + lc + 3 >= K) a.w = 0.f;
        }
        sa[lc][lr] = a.x; sa[lc + 1][lr] = a.y; sa[lc + 2][lr] = a.z; sa[lc + 3][lr] = a.w;
        sw[lc][lr] = w.x; sw[lc + 1][lr] = w.y; sw[lc + 2][lr] = w.z; sw[lc + 3][lr] = w.w;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kDepth; ++k) {
            const float4 av = *reinterpret_cast<const float4*>(&sa[k][ty * 4]);
            const float4 wv = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
            const float aa[4] = {av.x, av.y, av.z, av.w}, ww[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(aa[i], ww[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
            if (t >= T || n >= N) continue;
            if (e.what == Result::kGlu) {  // (N is even: both columns are there)
                if ((j & 1) == 0)
                    static_cast<float*>(e.cast)[(size_t)t * e.ld + n / 2] = clamped_glu(acc[i][j], acc[i][j | 1], e.limit, e.alpha);
                continue;
            }
            float* o = (e.what == Result::kCast ? static_cast<float*>(e.cast) : e.out) + (size_t)t * e.ld + n;
            if (e.what == Result::kAdd) *o += (e.scale ? e.scale[n] : 1.f) * acc[i][j];
            else *o = acc[i][j] + (e.bias ? e.bias[n] : 0.f);
        }
}

}  // namespace

cudaError_t gemm_f32(const float* A, int64_t lda, const float* W, int64_t ldw, int T, int N, int K,
                     const GemmEpilogue& e, cudaStream_t s) {
    gemm_f32_kernel<<<dim3((N + kTile - 1) / kTile, (T + kTile - 1) / kTile), 256, 0, s>>>(A, lda, W, ldw, T, N, K, e);
    return cudaGetLastError();
}

}  // namespace mkbh
