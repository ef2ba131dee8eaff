// Host-callable launchers of the hybrid models' kernels (one translation unit per group).
#pragma once
#include "hybrid_common.cuh"

namespace mkbh {

// What a matrix product does with its result: out[t, n] = acc + bias[n], or the residual
// update out[t, n] += scale[n] * acc.
struct GemmEpilogue {
    float* out;
    int64_t ld;
    const float* bias;   // may be NULL
    const float* scale;  // not NULL: residual update
};

// out[T, N] from A [T, lda] and W [N, ldw] (K columns of both, zero beyond, multiples of 8)
cudaError_t gemm_f32(const float* A, int64_t lda, const float* W, int64_t ldw, int T, int N, int K,
                     const GemmEpilogue& e, cudaStream_t s);
cudaError_t gemm_bf16(const bf16* A, int64_t lda, const bf16* W, int64_t ldw, int T, int N, int K,
                      const GemmEpilogue& e, int* status, cudaStream_t s);

// prefill kernels (template argument: element type of the model)
template <typename T>
struct Prefill {
    static cudaError_t embed(const MkbhGlobals& g, cudaStream_t s);
    // rows (NULL: all) of x -> normalised activations
    static cudaError_t norm(const float* x, const int32_t* rows, int n, int width, const float* w, float eps, T* out,
                            int64_t ld, cudaStream_t s);
    static cudaError_t poly_norm(const float* z, int64_t ldz, int n, int ff, const float* coeff, float eps, T* out,
                                 int64_t ld, cudaStream_t s);
    static cudaError_t delta(const MkbhGlobals& g, const MkbhLayer& L, T* out, int64_t ld, cudaStream_t s);
    static cudaError_t attention(const MkbhGlobals& g, const MkbhLayer& L, T* out, int64_t ld, cudaStream_t s);
};

// bf16 prefill attention on tensor cores, for head sizes it supports; writes columns [0, heads * vdim)
bool flash_supported(const MkbhLayer& L);
cudaError_t flash_attention(const MkbhGlobals& g, const MkbhLayer& L, const bf16* kc, const bf16* vc, bf16* out,
                            int64_t ldo, cudaStream_t s);

// decode: one persistent kernel
cudaError_t decode_launch(const MkbhGlobals& g, cudaStream_t s);

}  // namespace mkbh
