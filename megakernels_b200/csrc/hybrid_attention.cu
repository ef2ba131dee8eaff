// Prefill attention of the bf16 hybrid models over the cached rows, tiles of queries x 64 keys of
// one query head.  Scores, softmax and sums are fp32; the softmax weights enter the product with V
// as a bf16 pair (high and low part), so they keep 16 bits of mantissa.
//   flash_kernel         windowed differential attention: 64 queries; warps 0-3 carry the first map,
//                        warps 4-7 the second, over the same value tile.  The maps are combined,
//                        normalised and gated in the epilogue.
//   rotary_flash_kernel  one map, 128 queries: window, chunk or all keys; temperature and sink per
//                        head; values that turn with the position; keys in two pieces (latent).
#include "hybrid_kernels.h"

namespace mkbh {
namespace {

constexpr int kBQ = 64, kBKeys = 64;
constexpr int kFlashThreads = 256;

__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool live) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ float fast_exp2(float x) {  // arguments <= 0; tiny results flush to zero
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr)
                 : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr)
                 : "memory");
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct FlashArgs {
    const float* proj;
    int64_t ld, ldo;
    int n, pos0;
    MkbhLayer L;
    const bf16 *kc, *vc;
    bf16* out;
    float eps;
    int dp;  // dim padded to 16
};

struct FlashSmem {  // bf16 element offsets; row strides are odd multiples of 16 bytes
    int qs, vs, q, k, v, buf, total;
    __host__ __device__ FlashSmem(int dp, int ep) {
        qs = dp + 8;
        vs = ep + 8;
        q = 0;
        k = 2 * kBQ * qs;               // two buffers of [map][key][qs] and [key][vs]
        buf = 2 * kBKeys * qs + kBKeys * vs;
        v = k + 2 * kBKeys * qs;
        total = k + 2 * buf;
        const int merge = k + kBQ * (ep + 4) * 2;  // second map's rows as floats
        if (merge > total) total = merge;
    }
};

template <int EP>
__global__ void __launch_bounds__(kFlashThreads, EP <= 128 ? 2 : 1) flash_kernel(const FlashArgs a) {
    extern __shared__ __align__(128) bf16 sm[];
    const MkbhLayer& L = a.L;
    const int D = L.dim, E = L.vdim, G = L.kv_heads, dp = a.dp;
    const FlashSmem S(dp, EP);
    const int h = blockIdx.y, g = h / (L.heads / G), t0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kBQ;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int map = warp >> 2, r0 = (warp & 3) * 16;  // this warp's query rows
    const int nq = min(kBQ, a.n - t0);
    const int p0 = a.pos0 + t0, p1 = p0 + nq - 1;
    const int lo = max(0, p0 - L.window + 1), sinks = min(L.keep_first, lo);
    const int total = sinks + p1 - lo + 1;
    auto key_of = [&](int t) { return t < sinks ? t : lo + t - sinks; };
    // row of a key: the window is shorter than the ring, so it wraps at most once
    const int keep = L.cache_keep, ring = L.cache_ring, ring_lo = max(lo, keep), ring_row = (ring_lo - keep) % ring;
    auto row_of = [&](int j) {
        if (j < keep) return j;
        const int r = ring_row + (j - ring_lo);
        return keep + (r >= ring ? r - ring : r);
    };

    for (int i = tid; i < S.total / 8; i += kFlashThreads) reinterpret_cast<uint4*>(sm)[i] = make_uint4(0, 0, 0, 0);
    __syncthreads();  // padding columns stay zero
    for (int i = tid; i < nq * 2 * D; i += kFlashThreads) {
        const int r = i / (2 * D), c = i % (2 * D), m = c >= D;
        sm[S.q + (m * kBQ + r) * S.qs + c - m * D] = __float2bfloat16_rn(a.proj[(size_t)(t0 + r) * a.ld + h * 2 * D + c]);
    }
    const int kunits = D / 8, vunits = E / 8;
    auto fetch = [&](int tile, int buf) {
        const uint32_t kd = mkb::smem_u32(sm + S.k + buf * S.buf), vd = mkb::smem_u32(sm + S.v + buf * S.buf);
        for (int t = warp; t < kBKeys; t += kFlashThreads / 32) {  // one warp per key
            const int idx = tile * kBKeys + t;
            const bool live = idx < total;
            const size_t row = row_of(key_of(live ? idx : 0));
            const bf16 *ks = a.kc + (row * G + g) * 2 * D, *vs = a.vc + (row * G + g) * E;
            for (int u = lane; u < 2 * kunits + vunits; u += 32) {
                if (u < 2 * kunits) {
                    const int m = u >= kunits, c = (u - m * kunits) * 8;
                    cp16(kd + ((m * kBKeys + t) * S.qs + c) * 2, ks + m * D + c, live);
                } else {
                    const int c = (u - 2 * kunits) * 8;
                    cp16(vd + (t * S.vs + c) * 2, vs + c, live);
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    float o[EP / 8][4];
#pragma unroll
    for (int i = 0; i < EP / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
    float m_[2] = {-INFINITY, -INFINITY}, l_[2] = {0.f, 0.f};
    const float scale = L.scale * 1.4426950408889634f;
    const int row_pos[2] = {p0 + r0 + (lane >> 2), p0 + r0 + (lane >> 2) + 8};

    const int tiles = (total + kBKeys - 1) / kBKeys;
    fetch(0, 0);
    for (int tile = 0; tile < tiles; ++tile) {
        const int buf = tile & 1;
        if (tile + 1 < tiles) {
            fetch(tile + 1, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t qa = mkb::smem_u32(sm + S.q + (map * kBQ + r0 + (lane & 15)) * S.qs + (lane >> 4) * 8);
        // keys: lanes 0-7 / 8-15 the two k halves of keys 0..7, lanes 16-31 the same of keys 8..15
        const uint32_t ka = mkb::smem_u32(sm + S.k + buf * S.buf +
                                          (map * kBKeys + ((lane >> 4) << 3) + (lane & 7)) * S.qs + ((lane >> 3) & 1) * 8);
        float s[8][4];
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
        for (int k = 0; k < dp; k += 16) {
            uint32_t q[4];
            ldsm4(q, qa + k * 2);
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) {
                uint32_t b[4];
                ldsm4(b, ka + (nt * 16 * S.qs + k) * 2);
                mma(s[2 * nt], q, b[0], b[1]);
                mma(s[2 * nt + 1], q, b[2], b[3]);
            }
        }
        // mask only where the tile has keys that some query of the block does not see
        const int i0 = tile * kBKeys, i1 = min(i0 + kBKeys, total) - 1;
        const int j0 = key_of(i0), j1 = key_of(i1);
        const bool full = i1 == i0 + kBKeys - 1 && j1 <= p0 && (p1 - j0 < L.window || j1 < L.keep_first);
        if (!full) {
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int idx = i0 + i * 8 + (lane & 3) * 2 + (j & 1), key = key_of(idx), p = row_pos[j >> 1];
                    const bool see = idx < total && key <= p && (p - key < L.window || key < L.keep_first);
                    if (!see) s[i][j] = -INFINITY;
                }
        }
        float f[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float mx = m_[r];
#pragma unroll
            for (int i = 0; i < 8; ++i) mx = fmaxf(mx, fmaxf(s[i][2 * r], s[i][2 * r + 1]) * scale);
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            const float base = mx == -INFINITY ? 0.f : mx;
            f[r] = fast_exp2(m_[r] - base);
            m_[r] = mx;
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                s[i][2 * r] = fast_exp2(fmaf(s[i][2 * r], scale, -base));
                s[i][2 * r + 1] = fast_exp2(fmaf(s[i][2 * r + 1], scale, -base));
                sum += s[i][2 * r] + s[i][2 * r + 1];
            }
            l_[r] = l_[r] * f[r] + sum;
        }
        if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
            for (int i = 0; i < EP / 8; ++i) {
                o[i][0] *= f[0];
                o[i][1] *= f[0];
                o[i][2] *= f[1];
                o[i][3] *= f[1];
            }
        }
        // values: lanes 0-15 the 16 keys of columns 0..7, lanes 16-31 of columns 8..15
        const uint32_t va = mkb::smem_u32(sm + S.v + buf * S.buf + (lane & 15) * S.vs + (lane >> 4) * 8);
#pragma unroll
        for (int kt = 0; kt < 4; ++kt) {
            uint32_t hi[4], lw[4];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float y0 = s[2 * kt + (x >> 1)][(x & 1) * 2], y1 = s[2 * kt + (x >> 1)][(x & 1) * 2 + 1];
                hi[x] = mkb::pack_bf16x2(y0, y1);
                lw[x] = mkb::pack_bf16x2(y0 - mkb::bf16_lo(hi[x]), y1 - mkb::bf16_hi(hi[x]));
            }
#pragma unroll
            for (int nt = 0; nt < EP / 16; ++nt) {
                uint32_t b[4];
                ldsm4t(b, va + (kt * 16 * S.vs + nt * 16) * 2);
                mma(o[2 * nt], hi, b[0], b[1]);
                mma(o[2 * nt + 1], hi, b[2], b[3]);
                mma(o[2 * nt], lw, b[0], b[1]);
                mma(o[2 * nt + 1], lw, b[2], b[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l_[r] += __shfl_xor_sync(0xffffffffu, l_[r], 1);
        l_[r] += __shfl_xor_sync(0xffffffffu, l_[r], 2);
        l_[r] = l_[r] > 0.f ? 1.f / l_[r] : 0.f;  // rows beyond the portion have no keys
    }
    float* other = reinterpret_cast<float*>(sm + S.k);  // second map's rows (the tiles are done with)
    const int os = EP + 4;
    if (map == 1) {
#pragma unroll
        for (int i = 0; i < EP / 8; ++i)
#pragma unroll
            for (int r = 0; r < 2; ++r)
                *reinterpret_cast<float2*>(other + (r0 + (lane >> 2) + 8 * r) * os + i * 8 + (lane & 3) * 2) =
                    make_float2(o[i][2 * r] * l_[r], o[i][2 * r + 1] * l_[r]);
    }
    __syncthreads();
    if (map == 1) return;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = r0 + (lane >> 2) + 8 * r;
        float sq = 0.f;
#pragma unroll
        for (int i = 0; i < EP / 8; ++i) {
            const float2 b = *reinterpret_cast<const float2*>(other + row * os + i * 8 + (lane & 3) * 2);
            const float x = o[i][2 * r] * l_[r] - L.lambda * b.x, y = o[i][2 * r + 1] * l_[r] - L.lambda * b.y;
            o[i][2 * r] = x;
            o[i][2 * r + 1] = y;
            sq += x * x + y * y;
        }
        sq += __shfl_xor_sync(0xffffffffu, sq, 1);
        sq += __shfl_xor_sync(0xffffffffu, sq, 2);
        if (row >= nq) continue;  // (after the shuffles)
        const float fin = (1.f - L.diff) / sqrtf(sq / E + a.eps);
        const float* __restrict__ gate = a.proj + (size_t)(t0 + row) * a.ld + L.heads * 2 * D + h * E;
        bf16* __restrict__ dst = a.out + (size_t)(t0 + row) * a.ldo + h * E;
#pragma unroll
        for (int i = 0; i < EP / 8; ++i) {
            const int e = i * 8 + (lane & 3) * 2;
            if (e < E)  // E is a multiple of 8
                *reinterpret_cast<uint32_t*>(dst + e) =
                    mkb::pack_bf16x2(o[i][2 * r] * fin * sigmoid_f(__ldg(gate + e)), o[i][2 * r + 1] * fin * sigmoid_f(__ldg(gate + e + 1)));
        }
    }
}

template <int EP>
cudaError_t launch(const FlashArgs& a, cudaStream_t s) {
    static int set[64] = {};
    const int bytes = FlashSmem(a.dp, EP).total * 2;
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    if (set[dev & 63] < bytes) {
        e = cudaFuncSetAttribute(flash_kernel<EP>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
        if (e != cudaSuccess) return e;
        set[dev & 63] = bytes;
    }
    flash_kernel<EP><<<dim3((a.n + kBQ - 1) / kBQ, a.L.heads), kFlashThreads, bytes, s>>>(a);
    return cudaGetLastError();
}

// ---- one map ------------------------------------------------------------------------------- //
struct RotaryArgs {
    const bf16* query;
    int64_t ldq, ldo;
    int n, pos0;
    MkbhLayer L;
    KeySource<bf16> src;
    bf16* out;
    int dp;  // dot length padded to 16
};
constexpr int kRQ = 128;
struct RotarySmem {  // bf16 element offsets; row strides are odd multiples of 16 bytes
    int qs, vs, q, k, v, buf, total;
    __host__ __device__ RotarySmem(int dp, int ep) {
        qs = dp + 8;
        vs = ep + 8;
        q = 0;
        k = kRQ * qs;  // two buffers of [key][qs] and [key][vs]
        buf = kBKeys * (qs + vs);
        v = k + kBKeys * qs;
        total = k + 2 * buf;
    }
};

template <int EP>
__global__ void __launch_bounds__(kFlashThreads, EP <= 128 ? 2 : 1) rotary_flash_kernel(const RotaryArgs a) {
    extern __shared__ __align__(128) bf16 sm[];
    const MkbhLayer& L = a.L;
    const int A = a.src.split, B = a.src.rest, D = A + B, E = L.vdim, dp = a.dp;
    const RotarySmem S(dp, EP);
    const int h = blockIdx.y, g = h / a.src.per, t0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kRQ;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r0 = warp * 16;  // this warp's query rows
    const int nq = min(kRQ, a.n - t0), p0 = a.pos0 + t0, p1 = p0 + nq - 1;
    const int keep_first = L.chunk > 0 ? 0 : L.keep_first;
    auto first_key = [&](int p) { return L.chunk > 0 ? p - p % L.chunk : max(0, p - L.window + 1); };  // but for the kept ones
    const int lo = first_key(p0), sinks = min(keep_first, lo), total = sinks + p1 - lo + 1;
    auto key_of = [&](int t) { return t < sinks ? t : lo + t - sinks; };
    // row of a key: the visible stretch is shorter than the ring, so it wraps at most once
    const int keep = a.src.keep, ring = a.src.ring, ring_lo = max(lo, keep), ring_row = (ring_lo - keep) % ring;
    auto row_of = [&](int j) {
        if (j < keep) return j;
        const int r = ring_row + (j - ring_lo);
        return keep + (r >= ring ? r - ring : r);
    };

    for (int i = tid; i < S.total / 8; i += kFlashThreads) reinterpret_cast<uint4*>(sm)[i] = make_uint4(0, 0, 0, 0);
    __syncthreads();  // padding columns stay zero
    const int aunits = A / 8, kunits = D / 8, vunits = E / 8;
    for (int r = warp; r < nq; r += kFlashThreads / 32)
        for (int u = lane; u < kunits; u += 32)
            cp16(mkb::smem_u32(sm + S.q + r * S.qs + u * 8), a.query + (size_t)(t0 + r) * a.ldq + h * D + u * 8, true);
    auto fetch = [&](int tile, int buf) {
        const uint32_t kd = mkb::smem_u32(sm + S.k + buf * S.buf), vd = mkb::smem_u32(sm + S.v + buf * S.buf);
        for (int t = warp; t < kBKeys; t += kFlashThreads / 32) {  // one warp per key
            const int idx = tile * kBKeys + t;
            const bool live = idx < total;
            const size_t row = row_of(key_of(live ? idx : 0));
            const bf16 *ks = a.src.keys + row * a.src.key_ld + g * a.src.key_head, *vs = a.src.values + row * a.src.value_ld + g * a.src.value_head;
            for (int u = lane; u < kunits + vunits; u += 32) {
                if (u < kunits) cp16(kd + (t * S.qs + u * 8) * 2, u < aunits ? ks + u * 8 : a.src.shared + row * a.src.shared_ld + (u - aunits) * 8, live);
                else cp16(vd + (t * S.vs + (u - kunits) * 8) * 2, vs + (u - kunits) * 8, live);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    float o[EP / 8][4];
#pragma unroll
    for (int i = 0; i < EP / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
    // base 2; the sink is a key without a value that is there from the start
    const float log2e = 1.4426950408889634f, scale = L.scale * (L.temp ? __ldg(L.temp + h) : 1.f) * log2e;
    const float sink = L.sink ? __ldg(L.sink + h) * log2e : -INFINITY;
    float m_[2] = {sink, sink}, l_[2];
    l_[0] = l_[1] = L.sink && (lane & 3) == 0 ? 1.f : 0.f;
    const int row_pos[2] = {p0 + r0 + (lane >> 2), p0 + r0 + (lane >> 2) + 8};
    const int row_lo[2] = {first_key(row_pos[0]), first_key(row_pos[1])};
    const int warp_lo = first_key(p0 + r0), warp_hi = min(p0 + r0 + 15, p1), warp_last_lo = first_key(p0 + r0 + 15);

    const int tiles = (total + kBKeys - 1) / kBKeys;
    fetch(0, 0);
    for (int tile = 0; tile < tiles; ++tile) {
        const int buf = tile & 1;
        if (tile + 1 < tiles) {
            fetch(tile + 1, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int i0 = tile * kBKeys, i1 = min(i0 + kBKeys, total) - 1, j0 = key_of(i0), j1 = key_of(i1);
        // nothing here for any row of the warp?
        const bool none = p0 + r0 > p1 || j0 > warp_hi || (j1 < warp_lo && j0 >= keep_first);
        if (!none) {
            const uint32_t qa = mkb::smem_u32(sm + S.q + (r0 + (lane & 15)) * S.qs + (lane >> 4) * 8);
            // keys: lanes 0-7 / 8-15 the two k halves of keys 0..7, lanes 16-31 the same of keys 8..15
            const uint32_t ka = mkb::smem_u32(sm + S.k + buf * S.buf + (((lane >> 4) << 3) + (lane & 7)) * S.qs + ((lane >> 3) & 1) * 8);
            float s[8][4];
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
#pragma unroll 2
            for (int k = 0; k < dp; k += 16) {
                uint32_t q[4];
                ldsm4(q, qa + k * 2);
#pragma unroll
                for (int nt = 0; nt < 4; ++nt) {
                    uint32_t b[4];
                    ldsm4(b, ka + (nt * 16 * S.qs + k) * 2);
                    mma(s[2 * nt], q, b[0], b[1]);
                    mma(s[2 * nt + 1], q, b[2], b[3]);
                }
            }
            // mask only where the tile has keys that some row of the warp does not see
            const bool full = i1 == i0 + kBKeys - 1 && j1 <= p0 + r0 && (j0 >= warp_last_lo || j1 < keep_first);
            if (!full) {
#pragma unroll
                for (int i = 0; i < 8; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const int idx = i0 + i * 8 + (lane & 3) * 2 + (j & 1), key = key_of(idx);
                        const bool see = idx < total && key <= row_pos[j >> 1] && (key >= row_lo[j >> 1] || key < keep_first);
                        if (!see) s[i][j] = -INFINITY;
                    }
            }
            float f[2];
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                float mx = m_[r];
#pragma unroll
                for (int i = 0; i < 8; ++i) {  // (the scale may be negative: a temperature is any number)
                    s[i][2 * r] = s[i][2 * r] == -INFINITY ? -INFINITY : s[i][2 * r] * scale;
                    s[i][2 * r + 1] = s[i][2 * r + 1] == -INFINITY ? -INFINITY : s[i][2 * r + 1] * scale;
                    mx = fmaxf(mx, fmaxf(s[i][2 * r], s[i][2 * r + 1]));
                }
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                const float base = mx == -INFINITY ? 0.f : mx;
                f[r] = fast_exp2(m_[r] - base);
                m_[r] = mx;
                float sum = 0.f;
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    s[i][2 * r] = fast_exp2(s[i][2 * r] - base);
                    s[i][2 * r + 1] = fast_exp2(s[i][2 * r + 1] - base);
                    sum += s[i][2 * r] + s[i][2 * r + 1];
                }
                l_[r] = l_[r] * f[r] + sum;
            }
            if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
                for (int i = 0; i < EP / 8; ++i) {
                    o[i][0] *= f[0];
                    o[i][1] *= f[0];
                    o[i][2] *= f[1];
                    o[i][3] *= f[1];
                }
            }
            // values: lanes 0-15 the 16 keys of columns 0..7, lanes 16-31 of columns 8..15
            const uint32_t va = mkb::smem_u32(sm + S.v + buf * S.buf + (lane & 15) * S.vs + (lane >> 4) * 8);
#pragma unroll
            for (int kt = 0; kt < 4; ++kt) {
                uint32_t hi[4], lw[4];
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const float y0 = s[2 * kt + (x >> 1)][(x & 1) * 2], y1 = s[2 * kt + (x >> 1)][(x & 1) * 2 + 1];
                    hi[x] = mkb::pack_bf16x2(y0, y1);
                    lw[x] = mkb::pack_bf16x2(y0 - mkb::bf16_lo(hi[x]), y1 - mkb::bf16_hi(hi[x]));
                }
#pragma unroll
                for (int nt = 0; nt < EP / 16; ++nt) {
                    uint32_t b[4];
                    ldsm4t(b, va + (kt * 16 * S.vs + nt * 16) * 2);
                    mma(o[2 * nt], hi, b[0], b[1]);
                    mma(o[2 * nt + 1], hi, b[2], b[3]);
                    mma(o[2 * nt], lw, b[0], b[1]);
                    mma(o[2 * nt + 1], lw, b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l_[r] += __shfl_xor_sync(0xffffffffu, l_[r], 1);
        l_[r] += __shfl_xor_sync(0xffffffffu, l_[r], 2);
        const float inv = l_[r] > 0.f ? 1.f / l_[r] : 0.f;
        const int row = r0 + (lane >> 2) + 8 * r;
        if (row >= nq) continue;
        // neighbours, turned back by the query's angle
        const float2* turn = L.value_rope ? reinterpret_cast<const float2*>(L.value_rope) + (size_t)(p0 + row) * (E / 2) : nullptr;
        bf16* __restrict__ dst = a.out + (size_t)(t0 + row) * a.ldo + h * E;
#pragma unroll
        for (int i = 0; i < EP / 8; ++i) {
            const int e = i * 8 + (lane & 3) * 2;
            if (e >= E) continue;  // E is a multiple of 8
            float x = o[i][2 * r] * inv, y = o[i][2 * r + 1] * inv;
            if (turn != nullptr) {
                const float2 w = __ldg(turn + (e >> 1));
                const float z = x * w.x + y * w.y;
                y = y * w.x - x * w.y;
                x = z;
            }
            *reinterpret_cast<uint32_t*>(dst + e) = mkb::pack_bf16x2(x, y);
        }
    }
}

template <int EP>
cudaError_t launch_rotary(const RotaryArgs& a, cudaStream_t s) {
    static int set[64] = {};
    const int bytes = RotarySmem(a.dp, EP).total * 2;
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    if (set[dev & 63] < bytes) {
        e = cudaFuncSetAttribute(rotary_flash_kernel<EP>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
        if (e != cudaSuccess) return e;
        set[dev & 63] = bytes;
    }
    rotary_flash_kernel<EP><<<dim3((a.n + kRQ - 1) / kRQ, a.L.heads), kFlashThreads, bytes, s>>>(a);
    return cudaGetLastError();
}

}  // namespace

bool flash_supported(const MkbhLayer& L) { return L.dim % 8 == 0 && L.vdim % 8 == 0 && L.dim <= 128 && L.vdim <= 256; }

cudaError_t flash_attention(const MkbhGlobals& g, const MkbhLayer& L, const bf16* kc, const bf16* vc, bf16* out,
                            int64_t ldo, cudaStream_t s) {
    FlashArgs a{g.proj, pad8(L.in_rows), ldo, g.num_tokens, g.pos0, L, kc, vc, out, g.eps, (L.dim + 15) & ~15};
    if (L.vdim <= 32) return launch<32>(a, s);
    if (L.vdim <= 64) return launch<64>(a, s);
    if (L.vdim <= 128) return launch<128>(a, s);
    return launch<256>(a, s);
}

bool rotary_flash_supported(const MkbhLayer& L) {
    const int rest = L.mixer == MKBH_LATENT_ATTENTION ? L.rot_dim : 0, d = L.dim + rest;
    if (L.dim % 8 || rest % 8 || L.vdim % 8 || L.vdim > 256) return false;
    const int dp = (d + 15) & ~15, ep = L.vdim <= 32 ? 32 : L.vdim <= 64 ? 64 : L.vdim <= 128 ? 128 : 256;
    return RotarySmem(dp, ep).total * 2 <= 227 * 1024;
}

cudaError_t rotary_flash(const MkbhGlobals& g, const MkbhLayer& L, bf16* out, int64_t ldo, cudaStream_t s) {
    const KeySource<bf16> src = key_source<bf16>(g, L);
    const int d = src.split + src.rest;
    RotaryArgs a{static_cast<const bf16*>(g.query), pad8(L.heads * d), ldo, g.num_tokens, g.pos0, L, src, out, (d + 15) & ~15};
    if (L.vdim <= 32) return launch_rotary<32>(a, s);
    if (L.vdim <= 64) return launch_rotary<64>(a, s);
    if (L.vdim <= 128) return launch_rotary<128>(a, s);
    return launch_rotary<256>(a, s);
}

}  // namespace mkbh
