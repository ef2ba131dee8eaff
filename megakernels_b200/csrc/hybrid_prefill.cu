// Prefill kernels of the hybrid models other than the matrix products: embedding, norms, short
// convolutions, PolyNorm, the recurrence over a portion of tokens, and attention.
// Norms, scores, softmax weights, decays and the recurrent state are 32-bit in both builds.
#include "hybrid_kernels.h"

#include <type_traits>

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
            to_f(embed[(size_t)tok * width + i]) * scale + (pos != nullptr ? to_f(pos[(size_t)(pos0 + t) * width + i]) : 0.f);
}

// [residual stream | embedding] of every token
template <typename T>
__global__ void enter_kernel(const int32_t* __restrict__ tokens, int vocab, int width, float scale, const T* __restrict__ embed,
                             const float* __restrict__ x, T* __restrict__ out, int64_t ld) {
    const int t = blockIdx.x;
    int tok = tokens[t];
    tok = tok < 0 ? 0 : tok >= vocab ? vocab - 1 : tok;
    T* o = out + (size_t)t * ld;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        o[i] = from_f<T>(x[(size_t)t * width + i]);
        o[width + i] = from_f<T>(to_f(embed[(size_t)tok * width + i]) * scale);
    }
}

// ---- norms --------------------------------------------------------------------------- //
template <typename T>
__global__ void __launch_bounds__(kThreads) norm_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows,
                                                        int width, const float* __restrict__ w, float eps, bool centre,
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
    float mean = 0.f;
    if (centre) {
        block_sum<1, kThreads>(s, red);
        mean = s[0] / width;
    }
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

// The mixer's input h = N(x) w1, plus a causal convolution over time of its channels, and the input
// N(x) w2 of a feed-forward beside the mixer.  A block takes kNormTokens tokens and, before them,
// the inputs their convolution reaches back to (from the tokens of this portion, else from `hist`).
// The portion's last taps - 1 inputs go to `tail`, latest first.
constexpr int kNormTokens = 8;
template <typename T>
__global__ void __launch_bounds__(kThreads) canon_norm_kernel(const float* __restrict__ x, int n, int pos0, int width,
                                                              const float* __restrict__ w1, const float* __restrict__ w2,
                                                              float eps, bool centre, const float* __restrict__ taps_w, int taps,
                                                              const float* __restrict__ hist, float* __restrict__ tail,
                                                              T* __restrict__ out, T* __restrict__ out2, int64_t ld) {
    extern __shared__ __align__(16) float ring[];  // [taps][width]
    __shared__ float red[kThreads / 32];
    const int t0 = blockIdx.x * kNormTokens, t1 = min(n, t0 + kNormTokens), back = taps > 1 ? taps - 1 : 0;
    for (int t = t0 - back; t < t1; ++t) {
        float* h = ring + (taps > 0 ? (t + back) % taps : 0) * width;
        if (t < 0) {  // (every thread reads back only what it wrote itself)
            const int pos = pos0 + t;
            for (int i = threadIdx.x; i < width; i += kThreads) h[i] = pos >= 0 ? hist[(size_t)(pos % back) * width + i] : 0.f;
            continue;
        }
        const float* row = x + (size_t)t * width;
        float mean = 0.f, s[1] = {0.f};
        if (centre) {
            for (int i = threadIdx.x; i < width; i += kThreads) s[0] += row[i];
            block_sum<1, kThreads>(s, red);
            mean = s[0] / width;
            s[0] = 0.f;
        }
        for (int i = threadIdx.x; i < width; i += kThreads) s[0] += (row[i] - mean) * (row[i] - mean);
        block_sum<1, kThreads>(s, red);
        const float inv = 1.f / sqrtf(s[0] / width + eps);
        const bool live = t >= t0;
        for (int i = threadIdx.x; i < width; i += kThreads) {
            const float y = (row[i] - mean) * inv;
            float v = y * w1[i];
            if (taps > 0) {
                h[i] = v;
                if (live) {
                    float c = v;
                    for (int j = 0; j < taps; ++j) c = fmaf(taps_w[(size_t)j * width + i], ring[((t + back - (taps - 1) + j) % taps) * width + i], c);
                    if (n - 1 - t < back) tail[(size_t)(n - 1 - t) * width + i] = v;
                    v = c;
                }
            }
            if (live) {
                out[(size_t)t * ld + i] = from_f<T>(v);
                if (out2 != nullptr) out2[(size_t)t * ld + i] = from_f<T>(y * w2[i]);
            }
        }
    }
}

// The same for RMS norms, up to kTaps taps and widths that are multiples of 4: a warp per token for
// the norm, then four channels per thread, the convolution's inputs in registers.
template <typename T> struct Quad;
template <> struct Quad<float> { static __device__ __forceinline__ void put(float* o, float4 v) { *reinterpret_cast<float4*>(o) = v; } };
template <> struct Quad<bf16> {
    static __device__ __forceinline__ void put(bf16* o, float4 v) {
        *reinterpret_cast<uint2*>(o) = make_uint2(mkb::pack_bf16x2(v.x, v.y), mkb::pack_bf16x2(v.z, v.w));
    }
};
constexpr int kCanonTaps = 4;
template <typename T, int kT>
__global__ void __launch_bounds__(kThreads) canon_norm4_kernel(const float* __restrict__ x, int n, int pos0, int width,
                                                               const float* __restrict__ w1, const float* __restrict__ w2, float eps,
                                                               const float* __restrict__ taps_w, const float* __restrict__ hist,
                                                               float* __restrict__ tail, T* __restrict__ out, T* __restrict__ out2, int64_t ld) {
    constexpr int kBack = kT > 1 ? kT - 1 : 0, kRowsHere = kNormTokens + kBack;
    __shared__ float inv[kRowsHere];
    const int t0 = blockIdx.x * kNormTokens, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int i = warp; i < kRowsHere; i += kThreads / 32) {
        const int t = t0 - kBack + i;
        if (t < 0 || t >= n) continue;
        const float4* row = reinterpret_cast<const float4*>(x + (size_t)t * width);
        float s = 0.f;
#pragma unroll 8
        for (int c = lane; c < width / 4; c += 32) {
            const float4 v = row[c];
            s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        s = warp_sum(s);
        if (lane == 0) inv[i] = 1.f / sqrtf(s / width + eps);
    }
    __syncthreads();
    for (int c = 4 * threadIdx.x; c < width; c += 4 * kThreads) {
        const float4 a = *reinterpret_cast<const float4*>(w1 + c);
        const float4 b = out2 != nullptr ? *reinterpret_cast<const float4*>(w2 + c) : a;
        float4 tap[kT > 0 ? kT : 1], v[kRowsHere], h[kT > 0 ? kT : 1];  // h[k]: k tokens ago
#pragma unroll
        for (int k = 0; k < kT; ++k) {
            tap[k] = *reinterpret_cast<const float4*>(taps_w + (size_t)(kT - 1 - k) * width + c);
            h[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < kRowsHere; ++i) {
            const int t = t0 - kBack + i;
            v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (t >= 0 && t < n) v[i] = *reinterpret_cast<const float4*>(x + (size_t)t * width + c);
            else if (kBack > 0 && t < 0 && pos0 + t >= 0) v[i] = *reinterpret_cast<const float4*>(hist + (size_t)((pos0 + t) % (kBack > 0 ? kBack : 1)) * width + c);
        }
#pragma unroll
        for (int i = 0; i < kRowsHere; ++i) {
            const int t = t0 - kBack + i;
            if (t >= n) break;
            float4 y = v[i], in = y;  // (before the portion: the input itself)
            if (t >= 0) {
                const float f = inv[i];
                y = make_float4(y.x * f, y.y * f, y.z * f, y.w * f);
                in = make_float4(y.x * a.x, y.y * a.y, y.z * a.z, y.w * a.w);
            }
#pragma unroll
            for (int k = kT - 1; k > 0; --k) h[k] = h[k - 1];
            if (kT > 0) h[0] = in;
            if (i < kBack) continue;
            float4 o = in;
#pragma unroll
            for (int k = kT - 1; k >= 0; --k) {
                o.x = fmaf(tap[k].x, h[k].x, o.x);
                o.y = fmaf(tap[k].y, h[k].y, o.y);
                o.z = fmaf(tap[k].z, h[k].z, o.z);
                o.w = fmaf(tap[k].w, h[k].w, o.w);
            }
            if (kBack > 0 && n - 1 - t < kBack) *reinterpret_cast<float4*>(tail + (size_t)(n - 1 - t) * width + c) = in;
            Quad<T>::put(out + (size_t)t * ld + c, o);
            if (out2 != nullptr) Quad<T>::put(out2 + (size_t)t * ld + c, make_float4(y.x * b.x, y.y * b.y, y.z * b.z, y.w * b.w));
        }
    }
}

// After a portion: the last taps - 1 inputs of a convolution by position, and the sum of the next
// position's terms of earlier inputs.  `back(i)` is the input i tokens before the portion's end.
template <typename Back>
__device__ __forceinline__ void keep_channel(const float* w, float* hist, float* next, int taps, size_t ld, int n, int end, Back back) {
    // end: position of the portion's last token
    float s = 0.f;
    for (int i = 0; i < taps - 1 && i <= end; ++i) {
        const float v = i < n ? back(i) : hist[((end - i) % (taps - 1)) * ld];
        s = fmaf(w[(taps - 2 - i) * ld], v, s);
    }
    for (int i = 0; i < taps - 1 && i < n; ++i) hist[((end - i) % (taps - 1)) * ld] = back(i);
    *next = s;
}
__global__ void __launch_bounds__(kThreads) keep_inputs_kernel(const MkbhLayer L, int slot, int n, int pos0, int width,
                                                               const float* __restrict__ tail, const float* __restrict__ proj, int64_t ld) {
    const int ch = blockIdx.x * kThreads + threadIdx.x, end = pos0 + n - 1;
    if (L.canon_taps > 1 && ch < width)
        keep_channel(L.canon_w + ch, L.canon_hist + (size_t)slot * (L.canon_taps - 1) * width + ch,
                     L.canon_part + ((size_t)slot * 2 + ((end + 1) & 1)) * width + ch, L.canon_taps, width, n, end,
                     [&](int i) { return tail[(size_t)i * width + ch]; });
    if (L.conv_taps > 1 && ch < L.in_rows)
        keep_channel(L.conv_w + ch, L.conv_hist + (size_t)slot * (L.conv_taps - 1) * L.in_rows + ch,
                     L.conv_part + (size_t)slot * L.in_rows + ch, L.conv_taps, L.in_rows, n, end,
                     [&](int i) { return proj[(size_t)(n - 1 - i) * ld + ch]; });
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
// With c = sigmoid(a) / |k|^2 and q = k^T S (old state) a step is
//   S <- diag(w) S - (c k) q + k v^T.
// Per (token, head), one warp: replaces a by c, and writes what the scan's look-ahead needs,
//   alpha_t = k_(t+1) . (c_t k_t),  beta_t = k_(t+1) . k_t   (0 for the portion's last token).
// A warp takes 8 / R pairs at a time, R channels of each per lane (dim <= 32 R).
template <int R>
__global__ void __launch_bounds__(kThreads) delta_keys_kernel(float* __restrict__ proj, int64_t ld, int n, int heads,
                                                              int dim, float unit_eps, float* __restrict__ ab) {
    constexpr int P = 8 / R;
    const int HD = heads * dim, lane = threadIdx.x & 31;
    const int64_t first = ((int64_t)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5)) * P, total = (int64_t)n * heads;
    float x[P][R], y[P][R], av[P][R];
#pragma unroll
    for (int u = 0; u < P; ++u) {
        const int64_t item = first + u < total ? first + u : total - 1;
        const int t = (int)(item / heads), h = (int)(item % heads);
        const float* k = proj + (size_t)t * ld + HD + h * dim;
#pragma unroll
        for (int j = 0; j < R; ++j) {
            const int i = lane + 32 * j;
            const bool live = i < dim;
            x[u][j] = live ? k[i] : 0.f;
            y[u][j] = live && t + 1 < n ? k[ld + i] : 0.f;
            av[u][j] = live ? k[2 * HD + i] : 0.f;
        }
    }
#pragma unroll
    for (int u = 0; u < P; ++u) {
        const int64_t item = first + u;
        if (item >= total) break;  // uniform over the warp
        float kk = 0.f, beta = 0.f, alpha = 0.f;
#pragma unroll
        for (int j = 0; j < R; ++j) {
            const float s = sigmoid_f(av[u][j]);
            kk = fmaf(x[u][j], x[u][j], kk);
            beta = fmaf(x[u][j], y[u][j], beta);
            alpha = fmaf(x[u][j] * y[u][j], s, alpha);
            av[u][j] = s;
        }
        const float inv = 1.f / (warp_sum(kk) + unit_eps);
        alpha = warp_sum(alpha) * inv;
        beta = warp_sum(beta);
        float* a = proj + (size_t)(item / heads) * ld + 3 * HD + (item % heads) * dim;
#pragma unroll
        for (int j = 0; j < R; ++j)
            if (lane + 32 * j < dim) a[lane + 32 * j] = av[u][j] * inv;
        if (lane == 0) {
            ab[2 * item] = alpha;
            ab[2 * item + 1] = beta;
        }
    }
}

// Decays w = exp(-decay_scale * sigmoid(w2 tanh(w1) + w0)): a tile of 64 tokens x 64 channels of one head.
constexpr int kDecayTile = 64, kDecayStride = kDecayTile + 4;
__host__ __device__ inline int decay_smem(int rank) { return (kDecayTile * (rank | 1) + rank * kDecayStride) * 4; }
template <typename T>
__global__ void __launch_bounds__(kThreads) delta_decay_kernel(const float* __restrict__ proj, int64_t ld, int n, int HD,
                                                               int dim, int rank, const T* __restrict__ w2,
                                                               const float* __restrict__ w0, float decay_scale,
                                                               float* __restrict__ decay) {
    extern __shared__ __align__(16) float sm[];
    float* inner = sm;                         // [rank][64 tokens]
    float* wt = sm + rank * kDecayStride;      // [64 channels][rank | 1]
    const int t0 = blockIdx.x * kDecayTile, nt = min(kDecayTile, n - t0), ws = rank | 1;
    const int c0 = blockIdx.z * kDecayTile, nc = min(kDecayTile, dim - c0), col0 = blockIdx.y * dim + c0;
    for (int i = threadIdx.x; i < kDecayTile * rank; i += kThreads) {
        const int t = i / rank, r = i % rank;
        inner[r * kDecayStride + t] = t < nt ? tanhf(proj[(size_t)(t0 + t) * ld + 5 * HD + r]) : 0.f;
        wt[t * ws + r] = t < nc ? to_f(w2[(size_t)(col0 + t) * rank + r]) : 0.f;
    }
    __syncthreads();
    const int ch = threadIdx.x & 63, tg = (threadIdx.x >> 6) * 16;
    float acc[16];
#pragma unroll
    for (int j = 0; j < 16; ++j) acc[j] = 0.f;
    for (int r = 0; r < rank; ++r) {
        const float w = wt[ch * ws + r];
#pragma unroll
        for (int j = 0; j < 16; j += 4) {
            const float4 f = *reinterpret_cast<const float4*>(inner + r * kDecayStride + tg + j);
            acc[j] = fmaf(w, f.x, acc[j]);
            acc[j + 1] = fmaf(w, f.y, acc[j + 1]);
            acc[j + 2] = fmaf(w, f.z, acc[j + 2]);
            acc[j + 3] = fmaf(w, f.w, acc[j + 3]);
        }
    }
    if (ch >= nc) return;
    const float bias = w0[col0 + ch];
#pragma unroll
    for (int j = 0; j < 16; ++j)
        if (tg + j < nt) decay[(size_t)(t0 + tg + j) * HD + col0 + ch] = expf(-decay_scale * sigmoid_f(acc[j] + bias));
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
// state matrix are independent of each other.  Four warps compute: a warp holds 4 columns, 8 lanes
// per column; lane j of a column owns the key channels 32 m + 4 j + {0..3}, so that the broadcast
// reads of a token's vectors are conflict-free.  Four more warps keep the next chunk of tokens coming.
//
// The chain of a token is  q_t = k_t^T S_(t-1)  (a reduction over lanes)  ->  S_t.  One token of
// look-ahead halves it: with
//   q_(t+1) = (w_t k_(t+1))^T S_(t-1) - alpha_t q_t + beta_t v_t
// the reduction for token t + 1 starts from the state before token t.  Outputs are reduced for
// eight tokens at a time.
constexpr int kScanCols = 16;
constexpr int kScanThreads = 256;
template <int M>
__host__ __device__ constexpr int scan_tokens() { return M <= 2 ? 32 : M <= 4 ? 16 : 8; }
template <int M>
__host__ __device__ constexpr int scan_buf() {  // floats of one buffer
    return (scan_tokens<M>() + 1) * 4 * 32 * M + scan_tokens<M>() * (kScanCols + 2);
}
template <int M>
__host__ __device__ constexpr int scan_smem() { return 2 * scan_buf<M>() * 4; }

// A token's vectors as one lane needs them: decay, the NEXT token's key, removal rate, read vector.
template <int M>
struct ScanToken {
    float w[4 * M], kn[4 * M], c[4 * M], r[4 * M], v;
    float2 ab;
    __device__ __forceinline__ static void rows(float (&x)[4 * M], const float4* base) {
#pragma unroll
        for (int m = 0; m < M; ++m) {
            const float4 f = base[8 * m];
            x[4 * m] = f.x; x[4 * m + 1] = f.y; x[4 * m + 2] = f.z; x[4 * m + 3] = f.w;
        }
    }
    __device__ __forceinline__ void load(const float4* base, const float* vals, const float* abs_) {
        constexpr int Q = 8 * M;  // float4 per vector
        rows(w, base + 3 * Q);
        rows(kn, base + 5 * Q);
        rows(c, base + 2 * Q);
        rows(r, base);
        v = *vals;
        ab = *reinterpret_cast<const float2*>(abs_);
    }
};

template <int M>
__global__ void __launch_bounds__(kScanThreads, 1)
delta_scan_kernel(const float* __restrict__ proj, int64_t ld, int n, int heads, int dim, const float* __restrict__ decay,
                  const float* __restrict__ ab, float* __restrict__ state, int fresh, float* __restrict__ out) {
    constexpr int DP = 32 * M, TC = scan_tokens<M>(), BUF = scan_buf<M>();
    extern __shared__ __align__(16) float sm[];  // two of: [TC + 1][r k c w][DP], [TC][kScanCols], [TC][alpha beta]
    const int head = blockIdx.y, col0 = blockIdx.x * kScanCols, HD = heads * dim;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    for (int i = tid; i < 2 * BUF; i += kScanThreads) sm[i] = 0.f;  // padding channels stay zero
    __syncthreads();

    if (warp >= 4) {  // producers: warp 4 + q copies vector q of every token
        const int q = warp - 4, ptid = tid - 128;
        const float* src = q == 3 ? decay + head * dim : proj + head * dim + (q == 2 ? 3 : q) * HD;
        const int64_t stride = q == 3 ? HD : ld;
        const float *vsrc = proj + 2 * HD + head * dim + col0, *asrc = ab + head * 2;
        const bool wide = (dim % 4 == 0) && (HD % 4 == 0) && (ld % 4 == 0);
        const int units = wide ? dim / 4 : dim;               // copies per vector
        const int side = units < 32 ? 32 / units : 1;         // tokens side by side in a warp
        const int first = units < 32 ? lane / units : 0, u0 = units < 32 ? lane % units : lane;
        const int nc = min(kScanCols, dim - col0);
        for (int t0 = 0, buf = 0; t0 < n; t0 += TC, buf ^= 1) {
            if (t0 >= 2 * TC) __syncthreads();  // the buffer has been consumed
            float* b = sm + buf * BUF;
            const int nt = min(TC, n - t0), lim = q == 1 ? min(TC + 1, n - t0) : nt;  // keys: the next chunk's first as well
            if (first < side)
                for (int t = first; t < lim; t += side)
                    for (int u = u0; u < units; u += 32) {
                        const uint32_t dst = mkb::smem_u32(b + (t * 4 + q) * DP + u * (wide ? 4 : 1));
                        if (wide) cp_async16(dst, src + (t0 + t) * stride + u * 4);
                        else cp_async4(dst, src + (t0 + t) * stride + u);
                    }
            for (int t = lim; t < TC + (q == 1); ++t)  // beyond the portion: steps that change nothing
                for (int c = lane; c < dim; c += 32) b[(t * 4 + q) * DP + c] = q == 3 ? 1.f : 0.f;
            float *vals = b + (TC + 1) * 4 * DP, *abs_ = vals + TC * kScanCols;
            for (int i = ptid; i < TC * kScanCols; i += 128) {
                const int t = i / kScanCols, c = i % kScanCols;
                if (t < nt && c < nc) cp_async4(mkb::smem_u32(vals + i), vsrc + (t0 + t) * ld + c);
                else vals[i] = 0.f;
            }
            for (int i = ptid; i < TC * 2; i += 128) {
                if (i / 2 < nt) cp_async4(mkb::smem_u32(abs_ + i), asrc + (size_t)(t0 + i / 2) * heads * 2 + (i & 1));
                else abs_[i] = 0.f;
            }
            cp_async_commit();
            cp_async_wait<0>();
            __syncthreads();  // the chunk is there
        }
        return;
    }

    // Barriers of both sides, in order: chunk 0 there, chunk 1 there, chunk 0 consumed, chunk 2 there,
    // chunk 1 consumed, ...
    const int grp = lane & 7, lcol = warp * 4 + (lane >> 3), col = col0 + lcol, chunks = (n + TC - 1) / TC;
    const bool live = col < dim;
    float* S0 = state + ((size_t)head * dim + (live ? col : 0)) * dim;
    float S[4 * M];
#pragma unroll
    for (int i = 0; i < 4 * M; ++i) {
        const int ch = 32 * (i >> 2) + 4 * grp + (i & 3);
        S[i] = (!fresh && live && ch < dim) ? S0[ch] : 0.f;
    }
    float k[4 * M], q = 0.f;
    __syncthreads();  // chunk 0 is there
    for (int ci = 0; ci < chunks; ++ci) {
        const float* b = sm + (ci & 1) * BUF;
        const float4* vecs = reinterpret_cast<const float4*>(b) + grp;
        const float *vals = b + (TC + 1) * 4 * DP + lcol, *abs_ = b + (TC + 1) * 4 * DP + TC * kScanCols;
        if (ci == 0) {
            ScanToken<M>::rows(k, vecs + 8 * M);
#pragma unroll
            for (int i = 0; i < 4 * M; ++i) q = fmaf(k[i], S[i], q);
#pragma unroll
            for (int o = 1; o < 8; o <<= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
        }
        ScanToken<M> now, next;
        now.load(vecs, vals, abs_);
#pragma unroll 1
        for (int t8 = 0; t8 < TC; t8 += 8) {
            float op[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const int tn = j < 7 || t8 + 8 < TC ? t8 + j + 1 : 0;  // (the chunk's last token loads a dummy)
                next.load(vecs + tn * DP, vals + tn * kScanCols, abs_ + 2 * tn);
                float d[4] = {0.f, 0.f, 0.f, 0.f}, o[4] = {0.f, 0.f, 0.f, 0.f}, x[4 * M];
#pragma unroll
                for (int i = 0; i < 4 * M; ++i) {
                    S[i] *= now.w[i];
                    d[i & 3] = fmaf(now.kn[i], S[i], d[i & 3]);
                }
                float dd = (d[0] + d[1]) + (d[2] + d[3]);
                dd += __shfl_xor_sync(0xffffffffu, dd, 1);
#pragma unroll
                for (int i = 0; i < 4 * M; ++i) x[i] = fmaf(-now.c[i], q, now.v);
                dd += __shfl_xor_sync(0xffffffffu, dd, 2);
#pragma unroll
                for (int i = 0; i < 4 * M; ++i) S[i] = fmaf(k[i], x[i], S[i]);
                dd += __shfl_xor_sync(0xffffffffu, dd, 4);
#pragma unroll
                for (int i = 0; i < 4 * M; ++i) o[i & 3] = fmaf(now.r[i], S[i], o[i & 3]);
                op[j] = (o[0] + o[1]) + (o[2] + o[3]);
                q = fmaf(now.ab.y, now.v, fmaf(-now.ab.x, q, dd));
#pragma unroll
                for (int i = 0; i < 4 * M; ++i) k[i] = now.kn[i];
                now = next;
            }
            // eight sums over eight lanes in seven shuffles: lane j of a column ends up with token j
#pragma unroll
            for (int h = 4; h; h >>= 1)
#pragma unroll
                for (int j = 0; j < h; ++j) {
                    const bool up = grp & h;
                    const float keep = up ? op[j + h] : op[j], send = up ? op[j] : op[j + h];
                    op[j] = keep + __shfl_xor_sync(0xffffffffu, send, h);
                }
            const int t = ci * TC + t8 + grp;
            if (live && t < n) out[(size_t)t * HD + head * dim + col] = op[0];
        }
        if (ci + 1 < chunks) __syncthreads();  // chunk ci + 1 is there
        if (ci + 2 < chunks) __syncthreads();  // chunk ci has been consumed
    }
#pragma unroll
    for (int i = 0; i < 4 * M; ++i) {
        const int ch = 32 * (i >> 2) + 4 * grp + (i & 3);
        if (live && ch < dim) S0[ch] = S[i];
    }
}

// o of each head / its root mean square, times the norm weight, times sigmoid(g): one warp per
// (token, head), 8 / R of them at a time
template <typename T, int R>
__global__ void __launch_bounds__(kThreads) delta_gate_kernel(const float* __restrict__ o, const float* __restrict__ proj,
                                                              int64_t ld, int n, int heads, int dim,
                                                              const float* __restrict__ w, float eps,
                                                              T* __restrict__ out, int64_t ldo) {
    constexpr int P = 8 / R;
    const int HD = heads * dim, lane = threadIdx.x & 31;
    const int64_t first = ((int64_t)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5)) * P, total = (int64_t)n * heads;
    float v[P][R], x[P][R];
#pragma unroll
    for (int u = 0; u < P; ++u) {
        const int64_t item = first + u < total ? first + u : total - 1;
        const int t = (int)(item / heads), h = (int)(item % heads);
        const float *row = o + (size_t)t * HD + h * dim, *g = proj + (size_t)t * ld + 4 * HD + h * dim;
#pragma unroll
        for (int j = 0; j < R; ++j) {
            const int i = lane + 32 * j;
            v[u][j] = i < dim ? row[i] : 0.f;
            x[u][j] = i < dim ? g[i] : 0.f;
        }
    }
#pragma unroll
    for (int u = 0; u < P; ++u) {
        const int64_t item = first + u;
        if (item >= total) break;  // uniform over the warp
        const int t = (int)(item / heads), h = (int)(item % heads);
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < R; ++j) s = fmaf(v[u][j], v[u][j], s);
        const float inv = 1.f / sqrtf(warp_sum(s) / dim + eps);
        T* dst = out + (size_t)t * ldo + h * dim;
#pragma unroll
        for (int j = 0; j < R; ++j) {
            const int i = lane + 32 * j;
            if (i < dim) dst[i] = from_f<T>(v[u][j] * inv * w[h * dim + i] * sigmoid_f(x[u][j]));
        }
        if (h == heads - 1 && lane < pad8(HD) - HD) dst[dim + lane] = from_f<T>(0.f);
    }
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

// One CTA per (token, query head): scores of 128 keys at a time, both maps, online softmax.  The
// float build's attention, and the bf16 build's for head sizes hybrid_attention.cu does not take.
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
    const KeyRange keys(pos0 + t, L.window, L.keep_first, L.chunk);
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

// ---- rotary and latent attention ------------------------------------------------------------- //
// Operands of a portion.  A warp takes one vector (a query, key or value head; the latent, its
// rotated part) of kOpTokens tokens: convolution over time, norm, rotation of neighbours, and
// stores it as an element of the query buffer or as a cache row.
constexpr int kOpTokens = 8;
struct OperandArgs {
    const float* proj;
    int64_t ld, ldq;
    int n, pos0;
    MkbhLayer L;
    const float* hist;  // of the projection's convolution, this slot
    float eps;
    void *query, *kc, *vc;  // (cache bases of the slot)
    int qhead, qrest;       // entries of a query head, start of its rotated part
};
template <typename T, int J>
__device__ __forceinline__ void operand_vector(const OperandArgs& a, int t, int col, int len, const float* w, const float2* rope,
                                               int rot, T* dst) {
    const MkbhLayer& L = a.L;
    const int lane = threadIdx.x & 31, taps = L.conv_taps, pos = a.pos0 + t;
    float u[J][2], s = 0.f;
#pragma unroll
    for (int j = 0; j < J; ++j)
#pragma unroll
        for (int b = 0; b < 2; ++b) {
            const int i = 2 * (lane + 32 * j) + b, ch = col + i;
            float v = 0.f;
            if (i < len) {
                v = a.proj[(size_t)t * a.ld + ch];
                if (taps > 0) {
                    v *= L.conv_w[(size_t)(taps - 1) * L.in_rows + ch];
                    for (int k = 1; k < taps && k <= pos; ++k)  // k tokens ago
                        v = fmaf(L.conv_w[(size_t)(taps - 1 - k) * L.in_rows + ch],
                                 k <= t ? a.proj[(size_t)(t - k) * a.ld + ch] : a.hist[(size_t)((pos - k) % (taps - 1)) * L.in_rows + ch], v);
                }
            }
            u[j][b] = v;
            s = fmaf(v, v, s);
        }
    const float inv = w != nullptr ? 1.f / sqrtf(warp_sum(s) / len + a.eps) : 1.f;
#pragma unroll
    for (int j = 0; j < J; ++j) {
        const int i = 2 * (lane + 32 * j);
        if (i >= len) break;
        float x = u[j][0], y = u[j][1];
        if (w != nullptr) {
            x *= inv * w[i];
            if (i + 1 < len) y *= inv * w[i + 1];
        }
        if (i < rot) {
            const float2 r = rope[i >> 1];
            const float z = x * r.x - y * r.y;
            y = y * r.x + x * r.y;
            x = z;
        }
        dst[i] = from_f<T>(x);
        if (i + 1 < len) dst[i + 1] = from_f<T>(y);
    }
}
// The same for a run of tokens whose vector starts at an even column, with up to kTaps taps: every row
// is read once, as pairs; `dst` gives a token's place.  Columns len .. end of the place become zero.
constexpr int kTaps = 4;
template <typename T> struct Pair;
template <> struct Pair<float> { using type = float2; static __device__ __forceinline__ float2 make(float x, float y) { return make_float2(x, y); } };
template <> struct Pair<bf16> {
    using type = uint32_t;
    static __device__ __forceinline__ uint32_t make(float x, float y) { return mkb::pack_bf16x2(x, y); }
};
template <typename T, int J, bool kConv, typename Dst>
__device__ __forceinline__ void operand_run(const OperandArgs& a, int t0, int t1, int col, int len, const float* w, const float* rope, int rot,
                                            int end, Dst dst) {
    const MkbhLayer& L = a.L;
    const int lane = threadIdx.x & 31, taps = L.conv_taps;
    float2 tap[kConv ? kTaps : 1][J], norm[J], u[kConv ? kTaps : 1][J];  // tap k, u[k]: k tokens ago
#pragma unroll
    for (int j = 0; j < J; ++j) {
        const int i = 2 * (lane + 32 * j);
        const bool live = i < len;
        norm[j] = w != nullptr && live ? make_float2(w[i], w[i + 1]) : make_float2(1.f, 1.f);
        if constexpr (kConv) {
#pragma unroll
            for (int k = 0; k < kTaps; ++k) {
                const float* c = L.conv_w + (size_t)(taps - 1 - k) * L.in_rows + col + i;
                tap[k][j] = live && k < taps ? make_float2(c[0], c[1]) : make_float2(0.f, 0.f);
                const int t = t0 - k, pos = a.pos0 + t;  // (k = 0 is read in the loop)
                u[k][j] = make_float2(0.f, 0.f);
                if (!live || k == 0 || k >= taps) continue;
                if (t >= 0) u[k][j] = __ldg(reinterpret_cast<const float2*>(a.proj + (size_t)t * a.ld + col + i));
                else if (pos >= 0) {
                    const float* h = a.hist + (size_t)(pos % (taps - 1)) * L.in_rows + col + i;
                    u[k][j] = make_float2(h[0], h[1]);
                }
            }
        }
    }
#pragma unroll 4
    for (int t = t0; t < t1; ++t) {
        const float2* angles = reinterpret_cast<const float2*>(rope) + (size_t)(a.pos0 + t) * (rot / 2);
        float2 v[J], r[J];
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < J; ++j) {
            const int i = 2 * (lane + 32 * j);
            v[j] = i < len ? __ldg(reinterpret_cast<const float2*>(a.proj + (size_t)t * a.ld + col + i)) : make_float2(0.f, 0.f);
            r[j] = i < rot ? __ldg(angles + (i >> 1)) : make_float2(1.f, 0.f);
        }
#pragma unroll
        for (int j = 0; j < J; ++j) {
            if constexpr (kConv) {
                u[0][j] = v[j];
                float x = u[0][j].x * tap[0][j].x, y = u[0][j].y * tap[0][j].y;
#pragma unroll
                for (int k = 1; k < kTaps; ++k) x = fmaf(u[k][j].x, tap[k][j].x, x), y = fmaf(u[k][j].y, tap[k][j].y, y);
                v[j] = make_float2(x, y);
#pragma unroll
                for (int k = kTaps - 1; k > 0; --k) u[k][j] = u[k - 1][j];
            }
            s = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, s));
        }
        const float inv = w != nullptr ? 1.f / sqrtf(warp_sum(s) / len + a.eps) : 1.f;
        T* o = dst(t);
#pragma unroll
        for (int j = 0; j < J; ++j) {
            const int i = 2 * (lane + 32 * j);
            const float x = v[j].x * inv * norm[j].x, y = v[j].y * inv * norm[j].y;
            if (i < end) *reinterpret_cast<typename Pair<T>::type*>(o + i) = Pair<T>::make(x * r[j].x - y * r[j].y, y * r[j].x + x * r[j].y);
        }
        for (int i = 64 * J + 2 * lane; i < end; i += 64) *reinterpret_cast<typename Pair<T>::type*>(o + i) = Pair<T>::make(0.f, 0.f);
    }
}
// A vector of a run of tokens, by whatever path its size allows.
template <typename T, bool kConv, typename Dst>
__device__ __forceinline__ void operand_tokens(const OperandArgs& a, int t0, int t1, int col, int len, const float* w, const float* rope, int rot,
                                               int end, Dst dst) {
    const bool pairs = (col & 1) == 0 && (len & 1) == 0 && (rot == 0 || len >= rot) && (!kConv || a.L.conv_taps <= kTaps) &&
                       (reinterpret_cast<uint64_t>(dst(t0)) & (2 * sizeof(T) - 1)) == 0 && (reinterpret_cast<uint64_t>(dst(t0 + 1)) & (2 * sizeof(T) - 1)) == 0;
    if (pairs && len <= 64) return operand_run<T, 1, kConv>(a, t0, t1, col, len, w, rope, rot, end, dst);
    if (pairs && len <= 128) return operand_run<T, 2, kConv>(a, t0, t1, col, len, w, rope, rot, end, dst);
    if constexpr (!kConv) {
        if (pairs && len <= 256) return operand_run<T, 4, kConv>(a, t0, t1, col, len, w, rope, rot, end, dst);
        if (pairs) return operand_run<T, 8, kConv>(a, t0, t1, col, len, w, rope, rot, end, dst);
    }
    for (int t = t0; t < t1; ++t) {
        const float2* angles = reinterpret_cast<const float2*>(rope) + (size_t)(a.pos0 + t) * (rot / 2);
        if (len <= 256) operand_vector<T, 4>(a, t, col, len, w, angles, rot, dst(t));
        else operand_vector<T, 8>(a, t, col, len, w, angles, rot, dst(t));
        for (int i = len + (threadIdx.x & 31); i < end; i += 32) dst(t)[i] = from_f<T>(0.f);
    }
}
template <typename T, bool kLatent>
__global__ void __launch_bounds__(kThreads) rotary_operands_kernel(const OperandArgs a) {
    const MkbhLayer& L = a.L;
    const int task = blockIdx.y * (kThreads / 32) + (threadIdx.x >> 5), H = L.heads, G = L.kv_heads;
    if (task >= (kLatent ? H + 2 : H + 2 * G)) return;
    const int t0 = blockIdx.x * kOpTokens, t1 = min(a.n, t0 + kOpTokens);
    const size_t rows = L.cache_keep + L.cache_ring;
    auto query = [&](int h, int off) { return [=](int t) { return static_cast<T*>(a.query) + (size_t)t * a.ldq + h * a.qhead + off; }; };
    auto cache = [&](void* base, size_t first, int len, int off) {
        return [=](int t) { return static_cast<T*>(base) + (first + cache_row(a.pos0 + t, a.L.cache_keep, a.L.cache_ring)) * len + off; };
    };
    if constexpr (kLatent) {
        const int hd = L.dim + L.rot_dim, lr = latent_row(L);
        if (task < H) {
            operand_tokens<T, false>(a, t0, t1, task * hd, L.dim, nullptr, nullptr, 0, a.qrest, query(task, 0));
            operand_tokens<T, false>(a, t0, t1, task * hd + L.dim, L.rot_dim, nullptr, L.rope, L.rope_dims, a.qhead - a.qrest, query(task, a.qrest));
        } else if (task == H) {
            operand_tokens<T, false>(a, t0, t1, H * hd, L.rank, L.k_norm, nullptr, 0, L.rank, cache(a.kc, 0, lr, 0));
        } else {
            operand_tokens<T, false>(a, t0, t1, H * hd + L.rank, L.rot_dim, nullptr, L.rope, L.rope_dims, L.rot_dim, cache(a.kc, 0, lr, pad8(L.rank)));
        }
    } else {
        auto run = [&](auto conv) {
            constexpr bool kConv = decltype(conv)::value;
            if (task < H) {
                operand_tokens<T, kConv>(a, t0, t1, task * L.dim, L.dim, L.q_norm, L.rope, L.rope_dims, a.qhead, query(task, 0));
            } else if (task < H + G) {
                operand_tokens<T, kConv>(a, t0, t1, task * L.dim, L.dim, L.k_norm, L.rope, L.rope_dims, L.dim, cache(a.kc, (task - H) * rows, L.dim, 0));
            } else {
                const int g = task - H - G;
                operand_tokens<T, kConv>(a, t0, t1, (H + G) * L.dim + g * L.vdim, L.vdim, nullptr, L.value_rope, L.value_rope ? L.vdim : 0, L.vdim,
                                         cache(a.vc, g * rows, L.vdim, 0));
            }
        };
        if (L.conv_taps > 0) run(std::true_type{});
        else run(std::false_type{});
    }
}

// One CTA per (token, query head), 128 keys at a time, online softmax.  The float build's
// attention, and the bf16 build's for head sizes hybrid_attention.cu does not take.
template <typename T>
__global__ void __launch_bounds__(kAttnThreads) rotary_attention_kernel(const T* __restrict__ query, int64_t ldq, int pos0, const MkbhLayer L,
                                                                        const KeySource<T> src, T* __restrict__ out, int64_t ldo) {
    extern __shared__ float sm[];  // q [split + rest], p [128], o [vdim]
    __shared__ float red[kAttnThreads / 32];
    const int A = src.split, B = src.rest, E = L.vdim, H = L.heads;
    const int t = blockIdx.x, h = blockIdx.y, g = h / src.per, tid = threadIdx.x, pos = pos0 + t;
    float *q = sm, *p = sm + A + B, *o = p + kAttnThreads;
    for (int i = tid; i < A + B; i += kAttnThreads) q[i] = to_f(query[(size_t)t * ldq + h * (A + B) + i]);
    __syncthreads();
    const KeyRange keys(pos, L.window, L.keep_first, L.chunk);
    const float scale = L.scale * (L.temp ? L.temp[h] : 1.f);
    float m = L.sink ? L.sink[h] : -INFINITY, l = L.sink ? 1.f : 0.f, acc[kAttnMaxE] = {};
    for (int c0 = 0; c0 < keys.count; c0 += kAttnThreads) {
        const int nk = min(kAttnThreads, keys.count - c0);
        float s = -INFINITY;
        if (tid < nk) {
            const size_t row = cache_row(keys.key(c0 + tid), src.keep, src.ring);
            const T *k = src.keys + row * src.key_ld + g * src.key_head, *r = src.shared + row * src.shared_ld;
            float d = 0.f;
            for (int i = 0; i < A; ++i) d = fmaf(q[i], to_f(k[i]), d);
            for (int i = 0; i < B; ++i) d = fmaf(q[A + i], to_f(r[i]), d);
            s = d * scale;
        }
        float x = warp_max(s);
        if ((tid & 31) == 0) red[tid >> 5] = x;
        __syncthreads();
        x = m;
        for (int w = 0; w < kAttnThreads / 32; ++w) x = fmaxf(x, red[w]);
        const float f = expf(m - x);
        m = x;
        s = tid < nk ? expf(s - x) : 0.f;
        p[tid] = s;
        __syncthreads();
        float ps[1] = {s};
        block_sum<1, kAttnThreads>(ps, red);
        l = l * f + ps[0];
        for (int ei = 0; ei < kAttnMaxE; ++ei) {
            const int e = tid + ei * kAttnThreads;
            if (e >= E) break;
            float y = acc[ei] * f;
            for (int j = 0; j < nk; ++j)
                y = fmaf(p[j], to_f(src.values[(size_t)cache_row(keys.key(c0 + j), src.keep, src.ring) * src.value_ld + g * src.value_head + e]), y);
            acc[ei] = y;
        }
        __syncthreads();
    }
    for (int ei = 0; ei < kAttnMaxE; ++ei)
        if (tid + ei * kAttnThreads < E) o[tid + ei * kAttnThreads] = acc[ei] / l;
    __syncthreads();
    const float2* turn = L.value_rope ? reinterpret_cast<const float2*>(L.value_rope) + (size_t)pos * (E / 2) : nullptr;
    T* dst = out + (size_t)t * ldo + h * E;
    for (int e = tid; e < E; e += kAttnThreads) {
        float y = o[e];
        if (turn != nullptr) {  // back by the query's angle
            const float2 r = turn[e >> 1];
            y = y * r.x + (e & 1 ? -r.y : r.y) * o[e ^ 1];
        }
        dst[e] = from_f<T>(y);
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
    delta_scan_kernel<M><<<grid, kScanThreads, scan_smem<M>(), s>>>(
        g.proj, ld, g.num_tokens, L.heads, L.dim, g.decay, g.decay + (size_t)g.num_tokens * L.heads * L.dim, state,
        g.pos0 == 0, g.mixed);
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
cudaError_t Prefill<T>::enter(const MkbhGlobals& g, T* out, int64_t ld, cudaStream_t s) {
    enter_kernel<T><<<g.num_tokens, 256, 0, s>>>(g.tokens, g.vocab, g.width, g.embed_scale, static_cast<const T*>(g.embed), g.x, out, ld);
    return cudaGetLastError();
}
template <typename T>
cudaError_t Prefill<T>::norm(const MkbhGlobals& g, const int32_t* rows, int n, const float* w, T* out, int64_t ld, cudaStream_t s) {
    norm_kernel<T><<<n, kThreads, 0, s>>>(g.x, rows, g.width, w, g.eps, g.norm_kind == MKBH_LAYER_NORM, out, ld);
    return cudaGetLastError();
}
template <typename T>
cudaError_t Prefill<T>::canon_norm(const MkbhGlobals& g, const MkbhLayer& L, T* out, T* out2, int64_t ld, cudaStream_t s) {
    static int set[64] = {};
    const int n = g.num_tokens, smem = max(1, L.canon_taps) * g.width * 4;
    const float* hist = L.canon_hist + (L.canon_taps > 1 ? (size_t)g.slot * (L.canon_taps - 1) * g.width : 0);
    if (g.norm_kind == MKBH_RMS_NORM && g.width % 4 == 0 && L.canon_taps <= kCanonTaps) {
        auto go = [&](auto taps) {
            canon_norm4_kernel<T, decltype(taps)::value><<<(n + kNormTokens - 1) / kNormTokens, kThreads, 0, s>>>(
                g.x, n, g.pos0, g.width, L.norm1, L.norm2, g.eps, L.canon_w, hist, g.tail, out, out2, ld);
        };
        switch (L.canon_taps) {
            case 0: go(std::integral_constant<int, 0>{}); break;
            case 1: go(std::integral_constant<int, 1>{}); break;
            case 2: go(std::integral_constant<int, 2>{}); break;
            case 3: go(std::integral_constant<int, 3>{}); break;
            default: go(std::integral_constant<int, 4>{}); break;
        }
        return cudaGetLastError();
    }
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    if (smem > 48 * 1024 && set[dev & 63] < smem) {
        e = cudaFuncSetAttribute(canon_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return e;
        set[dev & 63] = smem;
    }
    canon_norm_kernel<T><<<(n + kNormTokens - 1) / kNormTokens, kThreads, smem, s>>>(
        g.x, n, g.pos0, g.width, L.norm1, L.norm2, g.eps, g.norm_kind == MKBH_LAYER_NORM, L.canon_w, L.canon_taps, hist, g.tail, out, out2, ld);
    return cudaGetLastError();
}
template <typename T>
cudaError_t Prefill<T>::keep_inputs(const MkbhGlobals& g, const MkbhLayer& L, cudaStream_t s) {
    const int channels = max(L.canon_taps > 1 ? g.width : 0, L.conv_taps > 1 ? L.in_rows : 0);
    keep_inputs_kernel<<<(channels + kThreads - 1) / kThreads, kThreads, 0, s>>>(L, g.slot, g.num_tokens, g.pos0, g.width, g.tail, g.proj,
                                                                                pad8(L.in_rows));
    return cudaGetLastError();
}
template <typename T>
cudaError_t Prefill<T>::rotary_operands(const MkbhGlobals& g, const MkbhLayer& L, cudaStream_t s) {
    const bool latent = L.mixer == MKBH_LATENT_ATTENTION;
    const int n = g.num_tokens, tasks = latent ? L.heads + 2 : L.heads + 2 * L.kv_heads;
    const size_t rows = (size_t)g.slot * (L.cache_keep + L.cache_ring);
    OperandArgs a{g.proj, pad8(L.in_rows), pad8(L.heads * query_head<T>(L)), n, g.pos0, L,
                  L.conv_hist + (L.conv_taps > 1 ? (size_t)g.slot * (L.conv_taps - 1) * L.in_rows : 0), g.eps, g.query,
                  static_cast<T*>(L.k_cache) + rows * (latent ? latent_row(L) : L.kv_heads * L.dim),
                  latent ? nullptr : static_cast<T*>(L.v_cache) + rows * L.kv_heads * L.vdim, query_head<T>(L), query_rest<T>(L)};
    const dim3 grid((n + kOpTokens - 1) / kOpTokens, (tasks + kThreads / 32 - 1) / (kThreads / 32));
    if (latent) rotary_operands_kernel<T, true><<<grid, kThreads, 0, s>>>(a);
    else rotary_operands_kernel<T, false><<<grid, kThreads, 0, s>>>(a);
    return cudaGetLastError();
}
template <typename T>
cudaError_t Prefill<T>::rotary_attention(const MkbhGlobals& g, const MkbhLayer& L, T* out, int64_t ldo, cudaStream_t s) {
    if constexpr (sizeof(T) == 2)
    {
        if (flash_tc_supported(L)) return flash_tc(g, L, out, ldo, s);
        if (rotary_flash_supported(L)) return rotary_flash(g, L, out, ldo, s);
    }
    const KeySource<T> src = key_source<T>(g, L);
    const int q = src.split + src.rest;
    rotary_attention_kernel<T><<<dim3(g.num_tokens, L.heads), kAttnThreads, (q + kAttnThreads + L.vdim) * 4, s>>>(
        static_cast<const T*>(g.query), pad8(L.heads * q), g.pos0, L, src, out, ldo);
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
    const int R = L.dim <= 64 ? 2 : L.dim <= 128 ? 4 : 8, per_block = kThreads / 32 * (8 / R);
    const int pairs = (int)(((int64_t)n * L.heads + per_block - 1) / per_block);
    float* ab = g.decay + (size_t)n * HD;
    if (R == 2) delta_keys_kernel<2><<<pairs, kThreads, 0, s>>>(g.proj, ld, n, L.heads, L.dim, L.unit_eps, ab);
    else if (R == 4) delta_keys_kernel<4><<<pairs, kThreads, 0, s>>>(g.proj, ld, n, L.heads, L.dim, L.unit_eps, ab);
    else delta_keys_kernel<8><<<pairs, kThreads, 0, s>>>(g.proj, ld, n, L.heads, L.dim, L.unit_eps, ab);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    const int smem = decay_smem(L.rank);
    if (smem > 48 * 1024) {
        e = cudaFuncSetAttribute(delta_decay_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return e;
    }
    delta_decay_kernel<T><<<dim3((n + kDecayTile - 1) / kDecayTile, L.heads, (L.dim + kDecayTile - 1) / kDecayTile), kThreads,
                            smem, s>>>(g.proj, ld, n, HD, L.dim, L.rank, static_cast<const T*>(L.decay_w2), L.decay_w0,
                                       L.decay_scale, g.decay);
    if ((e = cudaGetLastError()) != cudaSuccess) return e;
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
    if (R == 2) delta_gate_kernel<T, 2><<<pairs, kThreads, 0, s>>>(g.mixed, g.proj, ld, n, L.heads, L.dim, L.out_norm, g.eps, out, ldo);
    else if (R == 4) delta_gate_kernel<T, 4><<<pairs, kThreads, 0, s>>>(g.mixed, g.proj, ld, n, L.heads, L.dim, L.out_norm, g.eps, out, ldo);
    else delta_gate_kernel<T, 8><<<pairs, kThreads, 0, s>>>(g.mixed, g.proj, ld, n, L.heads, L.dim, L.out_norm, g.eps, out, ldo);
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
    if constexpr (sizeof(T) == 2)
        if (flash_supported(L)) return flash_attention(g, L, kc, vc, out, ldo, s);
    attention_kernel<T><<<dim3(n, L.heads), kAttnThreads, (2 * L.dim + 2 * kAttnThreads) * 4, s>>>(
        g.proj, ld, g.pos0, L, kc, vc, g.eps, out, ldo);
    return cudaGetLastError();
}

template struct Prefill<float>;
template struct Prefill<bf16>;

}  // namespace mkbh
