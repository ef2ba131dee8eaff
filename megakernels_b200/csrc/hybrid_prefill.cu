// Prefill kernels of the hybrid models other than the matrix products: embedding, layer norm,
// PolyNorm, the recurrence over a portion of tokens, and windowed differential attention.
// Norms, scores, softmax weights, decays and the recurrent state are 32-bit in both builds.
#include "hybrid_kernels.h"

namespace mkbh {
namespace {

constexpr int kThreads = 256;

// ---- embedding ------------------------------------------------------------------------- //
template <typename T>
__global__ void embed_kernel(const int32_t* __restrict__ tokens, int pos0, int vocab, int width, float scale,
                             const T* __restrict__ embed, const T* __restrict__ pos, float* __restrict__ x) {
    const int t = blockIdx.x;
    int tok = tokens[t];
    tok = tok < 0 ? 0 : tok >= vocab ? vocab - 1 : tok;  // ids are checked on the host; never read outside the table
    for (int i = threadIdx.x; i < width; i += blockDim.x)
        x[(size_t)t * width + i] =
            to_f(embed[(size_t)tok * width + i]) * scale + to_f(pos[(size_t)(pos0 + t) * width + i]);
}

// ---- layer norm --------------------------------------------------------------------------- //
template <typename T>
__global__ void __launch_bounds__(kThreads) norm_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows,
                                                        int width, const float* __restrict__ w, float eps,
                                                        T* __restrict__ out, int64_t ld) {
    __shared__ float red[kThreads / 32];
    const float* row = x + (size_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * width;
    T* o = out + (size_t)blockIdx.x * ld;
    constexpr int R = 8;  // elements kept in registers (wider rows are read again)
    float v[R], s[1] = {0.f};
#pragma unroll
    for (int k = 0; k < R; ++k) {
        const int i = threadIdx.x + k * kThreads;
        v[k] = i < width ? row[i] : 0.f;
        s[0] += v[k];
    }
    for (int i = threadIdx.x + R * kThreads; i < width; i += kThreads) s[0] += row[i];
    block_sum<1, kThreads>(s, red);
    const float mean = s[0] / width;
    s[0] = 0.f;
#pragma unroll
    for (int k = 0; k < R; ++k) {
        const float d = threadIdx.x + k * kThreads < width ? v[k] - mean : 0.f;
        s[0] += d * d;
    }
    for (int i = threadIdx.x + R * kThreads; i < width; i += kThreads) s[0] += (row[i] - mean) * (row[i] - mean);
    block_sum<1, kThreads>(s, red);
    const float inv = 1.f / sqrtf(s[0] / width + eps);
#pragma unroll
    for (int k = 0; k < R; ++k) {
        const int i = threadIdx.x + k * kThreads;
        if (i < width) o[i] = from_f<T>((v[k] - mean) * inv * w[i]);
    }
    for (int i = threadIdx.x + R * kThreads; i < width; i += kThreads) o[i] = from_f<T>((row[i] - mean) * inv * w[i]);
    for (int i = width + threadIdx.x; i < pad8(width); i += kThreads) o[i] = from_f<T>(0.f);
}

// ---- PolyNorm ----------------------------------------------------------------------------- //
template <typename T>
__global__ void __launch_bounds__(kThreads) poly_norm_kernel(const float* __restrict__ z, int64_t ldz, int ff, float ca,
                                                             float cb, float cc, float ce, float eps,
                                                             T* __restrict__ out, int64_t ld) {
    __shared__ float red[3 * kThreads / 32];
    const float* row = z + (size_t)blockIdx.x * ldz;
    T* o = out + (size_t)blockIdx.x * ld;
    float s[3] = {0.f, 0.f, 0.f};
    for (int i = threadIdx.x; i < ff; i += kThreads) {
        const float a = row[i] * row[i];
        s[0] += a;
        s[1] += a * a;
        s[2] += a * a * a;
    }
    block_sum<3, kThreads>(s, red);
    const float f1 = ca / sqrtf(s[0] / ff + eps), f2 = cb / sqrtf(s[1] / ff + eps), f3 = cc / sqrtf(s[2] / ff + eps);
    for (int i = threadIdx.x; i < ff; i += kThreads) {
        const float v = row[i];
        o[i] = from_f<T>(v * (f1 + v * (f2 + v * f3)) + ce);
    }
    for (int i = ff + threadIdx.x; i < pad8(ff); i += kThreads) o[i] = from_f<T>(0.f);
}

// ---- generalized delta rule ----------------------------------------------------------------- //
// The stacked projection of a token is [r | k | v | a | g | w1], heads * dim each but for w1.
// Replaces a by  c = sigmoid(a) / |k|^2  and writes the decays  w = exp(-decay_scale *
// sigmoid(w2 tanh(w1) + w0)), so that with q = k^T S the step is
//   S <- diag(w) S - (c k) q + k v^T.
constexpr int kPrepTokens = 16;
__global__ void __launch_bounds__(kThreads) delta_prep_kernel(float* __restrict__ proj, int64_t ld, int n, int HD,
                                                              int dim, int rank, const float* __restrict__ w2,
                                                              const float* __restrict__ w0, float decay_scale,
                                                              float unit_eps, float* __restrict__ decay) {
    extern __shared__ float sm[];  // [kPrepTokens][rank] tanh(w1), [kPrepTokens] 1 / |k|^2
    float* inner = sm;
    float* inv = sm + kPrepTokens * rank;
    const int head = blockIdx.y, t0 = blockIdx.x * kPrepTokens;
    const int nt = min(kPrepTokens, n - t0);
    for (int i = threadIdx.x; i < nt * rank; i += kThreads)
        inner[i] = tanhf(proj[(size_t)(t0 + i / rank) * ld + 5 * HD + i % rank]);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int t = warp; t < nt; t += kThreads / 32) {
        const float* k = proj + (size_t)(t0 + t) * ld + HD + head * dim;
        float s = 0.f;
        for (int i = lane; i < dim; i += 32) s += k[i] * k[i];
        s = warp_sum(s);
        if (lane == 0) inv[t] = 1.f / (s + unit_eps);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * dim; i += kThreads) {
        const int t = i / dim, col = head * dim + i % dim;
        const float* row = w2 + (size_t)col * rank;
        const float* in = inner + t * rank;
        float s = w0[col];
        for (int r = 0; r < rank; ++r) s += row[r] * in[r];
        decay[(size_t)(t0 + t) * HD + col] = expf(-decay_scale * sigmoid_f(s));
        float* a = proj + (size_t)(t0 + t) * ld + 3 * HD + col;
        *a = sigmoid_f(*a) * inv[t];
    }
}

__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// One CTA carries kScanCols value columns of one head through the portion: the columns of the
// state matrix are independent of each other.  A warp holds 4 columns, 8 lanes per column; lane
// group j of a column owns the key channels 32 m + 4 j + {0..3}, so that the broadcast reads of
// a token's vectors are conflict-free.
constexpr int kScanCols = 16;
constexpr int kScanThreads = 128;
template <int M>
__host__ __device__ constexpr int scan_tokens() { return M <= 2 ? 16 : 8; }
template <int M>
__host__ __device__ constexpr int scan_smem() { return 2 * scan_tokens<M>() * (4 * 32 * M + kScanCols) * 4; }

template <int M>
__global__ void __launch_bounds__(kScanThreads) delta_scan_kernel(const float* __restrict__ proj, int64_t ld, int n,
                                                                  int HD, int dim, const float* __restrict__ decay,
                                                                  float* __restrict__ state, int fresh,
                                                                  float* __restrict__ out) {
    constexpr int DP = 32 * M, TC = scan_tokens<M>();
    extern __shared__ __align__(16) float sm[];  // [2][TC][r k c w][DP], [2][TC][kScanCols]
    float* vec = sm;
    float* val = sm + 2 * TC * 4 * DP;
    const int head = blockIdx.y, col0 = blockIdx.x * kScanCols;
    const int tid = threadIdx.x, lane = tid & 31, grp = lane & 7;
    const int lcol = (tid >> 5) * 4 + (lane >> 3), col = col0 + lcol;
    const bool live = col < dim;
    for (int i = tid; i < 2 * TC * (4 * DP + kScanCols); i += kScanThreads) sm[i] = 0.f;  // padding channels stay zero
    float* S0 = state + (size_t)head * dim * dim;
    float S[4 * M];
#pragma unroll
    for (int m = 0; m < M; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 32 * m + 4 * grp + e;
            S[4 * m + e] = (!fresh && live && i < dim) ? S0[(size_t)i * dim + col] : 0.f;
        }
    __syncthreads();

    const float* src[4] = {proj + head * dim, proj + HD + head * dim, proj + 3 * HD + head * dim, decay + head * dim};
    const bool wide = (dim % 4 == 0) && (HD % 4 == 0) && (ld % 4 == 0);
    auto fetch = [&](int t0, int buf) {
        const int nt = min(TC, n - t0);
        const uint32_t dst = mkb::smem_u32(vec + buf * TC * 4 * DP);
        if (wide) {
            const int per = dim / 4;
            for (int i = tid; i < nt * 4 * per; i += kScanThreads) {
                const int t = i / (4 * per), q = i / per % 4, c = i % per;
                cp_async16(dst + ((t * 4 + q) * DP + c * 4) * 4, src[q] + (size_t)(t0 + t) * (q == 3 ? HD : ld) + c * 4);
            }
        } else {
            for (int i = tid; i < nt * 4 * dim; i += kScanThreads) {
                const int t = i / (4 * dim), q = i / dim % 4, c = i % dim;
                cp_async4(dst + ((t * 4 + q) * DP + c) * 4, src[q] + (size_t)(t0 + t) * (q == 3 ? HD : ld) + c);
            }
        }
        const uint32_t vdst = mkb::smem_u32(val + buf * TC * kScanCols);
        const int nc = min(kScanCols, dim - col0);
        for (int i = tid; i < nt * nc; i += kScanThreads)
            cp_async4(vdst + ((i / nc) * kScanCols + i % nc) * 4,
                      proj + (size_t)(t0 + i / nc) * ld + 2 * HD + head * dim + col0 + i % nc);
        cp_async_commit();
    };

    fetch(0, 0);
    for (int t0 = 0, buf = 0; t0 < n; t0 += TC, buf ^= 1) {
        if (t0 + TC < n) {
            fetch(t0 + TC, buf ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const int nt = min(TC, n - t0);
        for (int t = 0; t < nt; ++t) {
            const float4* base = reinterpret_cast<const float4*>(vec + (size_t)((buf * TC + t) * 4) * DP) + grp;
            float k[4 * M];
            float q0 = 0.f, q1 = 0.f;
#pragma unroll
            for (int m = 0; m < M; ++m) {
                const float4 f = base[DP / 4 + 8 * m];
                k[4 * m] = f.x; k[4 * m + 1] = f.y; k[4 * m + 2] = f.z; k[4 * m + 3] = f.w;
                q0 = fmaf(f.x, S[4 * m], q0);
                q1 = fmaf(f.y, S[4 * m + 1], q1);
                q0 = fmaf(f.z, S[4 * m + 2], q0);
                q1 = fmaf(f.w, S[4 * m + 3], q1);
            }
            float q = q0 + q1;
#pragma unroll
            for (int o = 1; o < 8; o <<= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
            const float v = val[(buf * TC + t) * kScanCols + lcol];
            float o0 = 0.f, o1 = 0.f;
#pragma unroll
            for (int m = 0; m < M; ++m) {
                const float4 c = base[2 * (DP / 4) + 8 * m], w = base[3 * (DP / 4) + 8 * m], r = base[8 * m];
                const float cc[4] = {c.x, c.y, c.z, c.w}, ww[4] = {w.x, w.y, w.z, w.w}, rr[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = 4 * m + e;
                    S[i] = fmaf(k[i], fmaf(-cc[e], q, v), ww[e] * S[i]);
                    if (e & 1) o1 = fmaf(rr[e], S[i], o1);
                    else o0 = fmaf(rr[e], S[i], o0);
                }
            }
            float o = o0 + o1;
#pragma unroll
            for (int d = 1; d < 8; d <<= 1) o += __shfl_xor_sync(0xffffffffu, o, d);
            if (grp == 0 && live) out[(size_t)(t0 + t) * HD + head * dim + col] = o;
        }
        __syncthreads();
    }
#pragma unroll
    for (int m = 0; m < M; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 32 * m + 4 * grp + e;
            if (live && i < dim) S0[(size_t)i * dim + col] = S[4 * m + e];
        }
}

// o of each head / its root mean square, times the norm weight, times sigmoid(g)
template <typename T>
__global__ void __launch_bounds__(kThreads) delta_gate_kernel(const float* __restrict__ o, const float* __restrict__ proj,
                                                              int64_t ld, int heads, int dim,
                                                              const float* __restrict__ w, float eps,
                                                              T* __restrict__ out, int64_t ldo) {
    const int HD = heads * dim, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float* row = o + (size_t)blockIdx.x * HD;
    const float* g = proj + (size_t)blockIdx.x * ld + 4 * HD;
    T* dst = out + (size_t)blockIdx.x * ldo;
    for (int h = warp; h < heads; h += kThreads / 32) {
        float s = 0.f;
        for (int i = lane; i < dim; i += 32) s += row[h * dim + i] * row[h * dim + i];
        const float inv = 1.f / sqrtf(warp_sum(s) / dim + eps);
        for (int i = lane; i < dim; i += 32) {
            const int c = h * dim + i;
            dst[c] = from_f<T>(row[c] * inv * w[c] * sigmoid_f(g[c]));
        }
    }
    for (int i = HD + threadIdx.x; i < pad8(HD); i += kThreads) dst[i] = from_f<T>(0.f);
}

// ---- windowed differential attention ---------------------------------------------------------- //
// keys and values of the portion -> their cache rows ([q | g | k | v] is the stacked projection)
template <typename T>
__global__ void kv_append_kernel(const float* __restrict__ proj, int64_t ld, int off, int kw, int vw, int pos0, int keep,
                                 int ring, T* __restrict__ kc, T* __restrict__ vc) {
    const float* src = proj + (size_t)blockIdx.x * ld + off;
    const size_t row = cache_row(pos0 + blockIdx.x, keep, ring);
    for (int i = threadIdx.x; i < kw + vw; i += blockDim.x) {
        if (i < kw) kc[row * kw + i] = from_f<T>(src[i]);
        else vc[row * vw + (i - kw)] = from_f<T>(src[i]);
    }
}

// One CTA per (token, query head): scores of 128 keys at a time, both maps, online softmax.
constexpr int kAttnThreads = 128;
constexpr int kAttnMaxE = 4;  // vdim <= 512
template <typename T>
__global__ void __launch_bounds__(kAttnThreads) attention_kernel(const float* __restrict__ proj, int64_t ld, int pos0,
                                                                 MkbhLayer L, const T* __restrict__ kc,
                                                                 const T* __restrict__ vc, float eps, T* __restrict__ out,
                                                                 int64_t ldo) {
    extern __shared__ float sm[];  // q [2 dim], p [2][128]
    __shared__ float red[2 * kAttnThreads / 32];
    const int D = L.dim, E = L.vdim, G = L.kv_heads, H = L.heads;
    const int t = blockIdx.x, h = blockIdx.y, g = h / (H / G), tid = threadIdx.x;
    float* q = sm;
    float* p = sm + 2 * D;
    const float* row = proj + (size_t)t * ld;
    // (q takes the precision of the activations it would have had as a stored tensor)
    for (int i = tid; i < 2 * D; i += kAttnThreads) q[i] = to_f(from_f<T>(row[h * 2 * D + i]));
    __syncthreads();
    const KeyRange keys(pos0 + t, L.window, L.keep_first);
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, acc[2][kAttnMaxE] = {};
    for (int c0 = 0; c0 < keys.count; c0 += kAttnThreads) {
        const int nk = min(kAttnThreads, keys.count - c0);
        float s[2] = {-INFINITY, -INFINITY};
        if (tid < nk) {
            const T* k = kc + ((size_t)cache_row(keys.key(c0 + tid), L.cache_keep, L.cache_ring) * G + g) * 2 * D;
            for (int b = 0; b < 2; ++b) {
                float d = 0.f;
                for (int i = 0; i < D; ++i) d = fmaf(q[b * D + i], to_f(k[b * D + i]), d);
                s[b] = d * L.scale;
            }
        }
        for (int b = 0; b < 2; ++b) {
            float x = warp_max(s[b]);
            if ((tid & 31) == 0) red[b * (kAttnThreads / 32) + (tid >> 5)] = x;
        }
        __syncthreads();
        float f[2];
        for (int b = 0; b < 2; ++b) {
            float x = m[b];
            for (int w = 0; w < kAttnThreads / 32; ++w) x = fmaxf(x, red[b * (kAttnThreads / 32) + w]);
            f[b] = expf(m[b] - x);
            m[b] = x;
            s[b] = tid < nk ? expf(s[b] - x) : 0.f;
            p[b * kAttnThreads + tid] = s[b];
        }
        __syncthreads();
        float ps[2] = {s[0], s[1]};
        block_sum<2, kAttnThreads>(ps, red);
        for (int b = 0; b < 2; ++b) l[b] = l[b] * f[b] + ps[b];
        for (int ei = 0; ei < kAttnMaxE; ++ei) {
            const int e = tid + ei * kAttnThreads;
            if (e >= E) break;
            float a0 = acc[0][ei] * f[0], a1 = acc[1][ei] * f[1];
            for (int j = 0; j < nk; ++j) {
                const float v = to_f(vc[((size_t)cache_row(keys.key(c0 + j), L.cache_keep, L.cache_ring) * G + g) * E + e]);
                a0 = fmaf(p[j], v, a0);
                a1 = fmaf(p[kAttnThreads + j], v, a1);
            }
            acc[0][ei] = a0;
            acc[1][ei] = a1;
        }
        __syncthreads();
    }
    float sq[1] = {0.f};
    for (int ei = 0; ei < kAttnMaxE; ++ei) {
        const float o = tid + ei * kAttnThreads < E ? acc[0][ei] / l[0] - L.lambda * (acc[1][ei] / l[1]) : 0.f;
        acc[0][ei] = o;
        sq[0] += o * o;
    }
    block_sum<1, kAttnThreads>(sq, red);
    const float f = (1.f - L.diff) / sqrtf(sq[0] / E + eps);
    const float* gate = row + H * 2 * D + h * E;
    T* dst = out + (size_t)t * ldo + h * E;
    for (int ei = 0; ei < kAttnMaxE; ++ei) {
        const int e = tid + ei * kAttnThreads;
        if (e < E) dst[e] = from_f<T>(acc[0][ei] * f * sigmoid_f(gate[e]));
    }
    if (h == 0)
        for (int i = H * E + tid; i < pad8(H * E); i += kAttnThreads) out[(size_t)t * ldo + i] = from_f<T>(0.f);
}

template <int M>
cudaError_t launch_scan(const MkbhGlobals& g, const MkbhLayer& L, int64_t ld, float* state, cudaStream_t s) {
    static bool set[64] = {};
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    if (!set[dev & 63]) {
        e = cudaFuncSetAttribute(delta_scan_kernel<M>, cudaFuncAttributeMaxDynamicSharedMemorySize, scan_smem<M>());
        if (e != cudaSuccess) return e;
        set[dev & 63] = true;
    }
    dim3 grid((L.dim + kScanCols - 1) / kScanCols, L.heads);
    delta_scan_kernel<M><<<grid, kScanThreads, scan_smem<M>(), s>>>(g.proj, ld, g.num_tokens, L.heads * L.dim, L.dim,
                                                                   g.decay, state, g.pos0 == 0, g.mixed);
    return cudaGetLastError();
}

}  // namespace

template <typename T>
cudaError_t Prefill<T>::embed(const MkbhGlobals& g, cudaStream_t s) {
    embed_kernel<T><<<g.num_tokens, 256, 0, s>>>(g.tokens, g.pos0, g.vocab, g.width, g.embed_scale,
                                                 static_cast<const T*>(g.embed), static_cast<const T*>(g.pos), g.x);
    return cudaGetLastError();
}
template <typename T>
cudaError_t Prefill<T>::norm(const float* x, const int32_t* rows, int n, int width, const float* w, float eps, T* out,
                             int64_t ld, cudaStream_t s) {
    norm_kernel<T><<<n, kThreads, 0, s>>>(x, rows, width, w, eps, out, ld);
    return cudaGetLastError();
}
template <typename T>
cudaError_t Prefill<T>::poly_norm(const float* z, int64_t ldz, int n, int ff, const float* c, float eps, T* out,
                                  int64_t ld, cudaStream_t s) {
    poly_norm_kernel<T><<<n, kThreads, 0, s>>>(z, ldz, ff, c[0], c[1], c[2], c[3], eps, out, ld);
    return cudaGetLastError();
}
template <typename T>
cudaError_t Prefill<T>::delta(const MkbhGlobals& g, const MkbhLayer& L, T* out, int64_t ldo, cudaStream_t s) {
    const int n = g.num_tokens, HD = L.heads * L.dim;
    const int64_t ld = pad8(L.in_rows);
    const int smem = kPrepTokens * (L.rank + 1) * 4;
    delta_prep_kernel<<<dim3((n + kPrepTokens - 1) / kPrepTokens, L.heads), kThreads, smem, s>>>(
        g.proj, ld, n, HD, L.dim, L.rank, L.decay_w2, L.decay_w0, L.decay_scale, L.unit_eps, g.decay);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    float* state = L.state + (size_t)g.slot * HD * L.dim;
    switch ((L.dim + 31) / 32) {
        case 1: e = launch_scan<1>(g, L, ld, state, s); break;
        case 2: e = launch_scan<2>(g, L, ld, state, s); break;
        case 3: e = launch_scan<3>(g, L, ld, state, s); break;
        case 4: e = launch_scan<4>(g, L, ld, state, s); break;
        case 5: case 6: e = launch_scan<6>(g, L, ld, state, s); break;
        case 7: case 8: e = launch_scan<8>(g, L, ld, state, s); break;
        default: return cudaErrorInvalidValue;
    }
    if (e != cudaSuccess) return e;
    delta_gate_kernel<T><<<n, kThreads, 0, s>>>(g.mixed, g.proj, ld, L.heads, L.dim, L.out_norm, g.eps, out, ldo);
    return cudaGetLastError();
}
template <typename T>
cudaError_t Prefill<T>::attention(const MkbhGlobals& g, const MkbhLayer& L, T* out, int64_t ldo, cudaStream_t s) {
    const int n = g.num_tokens, kw = L.kv_heads * 2 * L.dim, vw = L.kv_heads * L.vdim;
    const int64_t ld = pad8(L.in_rows);
    const size_t rows = (size_t)g.slot * (L.cache_keep + L.cache_ring);
    T* kc = static_cast<T*>(L.k_cache) + rows * kw;
    T* vc = static_cast<T*>(L.v_cache) + rows * vw;
    if (L.owns_kv) {
        kv_append_kernel<T><<<n, 256, 0, s>>>(g.proj, ld, L.heads * (2 * L.dim + L.vdim), kw, vw, g.pos0, L.cache_keep,
                                              L.cache_ring, kc, vc);
        cudaError_t e = cudaGetLastError();
        if (e != cudaSuccess) return e;
    }
    attention_kernel<T><<<dim3(n, L.heads), kAttnThreads, (2 * L.dim + 2 * kAttnThreads) * 4, s>>>(
        g.proj, ld, g.pos0, L, kc, vc, g.eps, out, ldo);
    return cudaGetLastError();
}

template struct Prefill<float>;
template struct Prefill<bf16>;

}  // namespace mkbh
