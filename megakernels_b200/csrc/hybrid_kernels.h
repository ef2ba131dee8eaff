// Host-callable launchers of the hybrid models' kernels (one translation unit per group).
#pragma once
#include "hybrid_common.cuh"

namespace mkbh {

// What a matrix product does with its result.
enum class Result {
    kStore,  // out[t, n] = acc + bias[n]
    kAdd,    // out[t, n] += scale[n] * acc (the residual stream)
    kCast,   // cast[t, n] = acc in the model dtype
    kGlu,    // cast[t, n / 2] = clamped gated unit of columns n (gate) and n + 1
};
struct GemmEpilogue {
    Result what;
    float* out;
    void* cast;
    int64_t ld;
    const float* bias;   // kStore; may be NULL
    const float* scale;  // kAdd; NULL: 1
    float limit, alpha;  // kGlu
    static GemmEpilogue store(float* out, int64_t ld, const float* bias) { return {Result::kStore, out, nullptr, ld, bias, nullptr, 0.f, 0.f}; }
    static GemmEpilogue add(float* out, int64_t ld, const float* scale) { return {Result::kAdd, out, nullptr, ld, nullptr, scale, 0.f, 0.f}; }
    static GemmEpilogue to(void* out, int64_t ld) { return {Result::kCast, nullptr, out, ld, nullptr, nullptr, 0.f, 0.f}; }
    static GemmEpilogue glu(void* out, int64_t ld, float limit, float alpha) { return {Result::kGlu, nullptr, out, ld, nullptr, nullptr, limit, alpha}; }
};

// out[T, N] from A [T, lda] and W [N, ldw], K columns of both (rows 16-byte aligned)
cudaError_t gemm_f32(const float* A, int64_t lda, const float* W, int64_t ldw, int T, int N, int K,
                     const GemmEpilogue& e, cudaStream_t s);
cudaError_t gemm_bf16(const bf16* A, int64_t lda, const bf16* W, int64_t ldw, int T, int N, int K,
                      const GemmEpilogue& e, int* status, cudaStream_t s);

// prefill kernels (template argument: element type of the model)
template <typename T>
struct Prefill {
    static cudaError_t embed(const MkbhGlobals& g, cudaStream_t s);
    // [residual stream | embedding]
    static cudaError_t enter(const MkbhGlobals& g, T* out, int64_t ld, cudaStream_t s);
    // rows (NULL: all) of x -> normalised activations
    static cudaError_t norm(const MkbhGlobals& g, const int32_t* rows, int n, const float* w, T* out, int64_t ld, cudaStream_t s);
    // the mixer's input (norm, convolution) and, if `out2`, the feed-forward's beside it
    static cudaError_t canon_norm(const MkbhGlobals& g, const MkbhLayer& L, T* out, T* out2, int64_t ld, cudaStream_t s);
    // inputs that later tokens' convolutions need
    static cudaError_t keep_inputs(const MkbhGlobals& g, const MkbhLayer& L, cudaStream_t s);
    static cudaError_t poly_norm(const float* z, int64_t ldz, int n, int ff, const float* coeff, float eps, T* out,
                                 int64_t ld, cudaStream_t s);
    static cudaError_t delta(const MkbhGlobals& g, const MkbhLayer& L, T* out, int64_t ld, cudaStream_t s);
    static cudaError_t attention(const MkbhGlobals& g, const MkbhLayer& L, T* out, int64_t ld, cudaStream_t s);
    // rotary and latent attention: operands (convolution, norm, rotation, cache rows), then the attention
    static cudaError_t rotary_operands(const MkbhGlobals& g, const MkbhLayer& L, cudaStream_t s);
    static cudaError_t rotary_attention(const MkbhGlobals& g, const MkbhLayer& L, T* out, int64_t ld, cudaStream_t s);
};

// bf16 prefill attention on tensor cores, for head sizes it supports; writes columns [0, heads * vdim)
bool flash_supported(const MkbhLayer& L);
cudaError_t flash_attention(const MkbhGlobals& g, const MkbhLayer& L, const bf16* kc, const bf16* vc, bf16* out,
                            int64_t ldo, cudaStream_t s);

// Where rotary and latent attention find a position's key and value: the key is `split` entries at
// keys[row][head] and, for a latent, `rest` more that all heads share.
template <typename T>
struct KeySource {
    const T *keys, *shared, *values;
    int64_t key_ld, shared_ld, value_ld;  // elements between rows
    int64_t key_head, value_head;         // elements between key/value heads
    int split, rest, per;                 // query heads per key/value head
    int keep, ring;
};
template <typename T>
inline KeySource<T> key_source(const MkbhGlobals& g, const MkbhLayer& L) {
    const size_t row0 = (size_t)g.slot * (L.cache_keep + L.cache_ring);
    if (L.mixer == MKBH_LATENT_ATTENTION) {
        const int64_t ld = pad8(L.heads * (L.dim + L.vdim)), lr = latent_row(L);
        const T* keys = static_cast<const T*>(g.keys);
        return {keys, static_cast<const T*>(L.k_cache) + row0 * lr + pad8(L.rank), keys + L.heads * L.dim, ld, lr, ld, L.dim, L.vdim,
                L.dim, L.rot_dim, 1, 0, L.cache_ring};
    }
    const int64_t rows = L.cache_keep + L.cache_ring;
    return {static_cast<const T*>(L.k_cache) + row0 * L.kv_heads * L.dim, nullptr, static_cast<const T*>(L.v_cache) + row0 * L.kv_heads * L.vdim,
            L.dim, 0, L.vdim, rows * L.dim, rows * L.vdim, L.dim, 0, L.heads / L.kv_heads, L.cache_keep, L.cache_ring};
}
// tcgen05 (sizes it supports), mma.sync (more sizes)
bool flash_tc_supported(const MkbhLayer& L);
// Entries of a query head, and where its rotated part (latent) starts: the tensor-core kernel reads
// whole slabs of 64 columns, zero beyond either part.
template <typename T>
inline int query_rest(const MkbhLayer& L) { return sizeof(T) == 2 && flash_tc_supported(L) ? (L.dim + 63) / 64 * 64 : L.dim; }
template <typename T>
inline int query_head(const MkbhLayer& L) {
    const int rest = L.mixer == MKBH_LATENT_ATTENTION ? L.rot_dim : 0;
    return query_rest<T>(L) + (sizeof(T) == 2 && flash_tc_supported(L) ? (rest + 63) / 64 * 64 : rest);
}
cudaError_t flash_tc(const MkbhGlobals& g, const MkbhLayer& L, bf16* out, int64_t ldo, cudaStream_t s);
bool rotary_flash_supported(const MkbhLayer& L);
cudaError_t rotary_flash(const MkbhGlobals& g, const MkbhLayer& L, bf16* out, int64_t ldo, cudaStream_t s);

// decode: one persistent kernel, built per set of mechanisms
template <int kFeatures>
cudaError_t decode_build(const MkbhGlobals& g, cudaStream_t s);
template <> cudaError_t decode_build<1>(const MkbhGlobals& g, cudaStream_t s);
template <> cudaError_t decode_build<2>(const MkbhGlobals& g, cudaStream_t s);
template <> cudaError_t decode_build<3>(const MkbhGlobals& g, cudaStream_t s);
cudaError_t decode_launch(const MkbhGlobals& g, cudaStream_t s);

}  // namespace mkbh
