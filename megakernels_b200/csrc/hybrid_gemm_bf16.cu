// bf16 matrix product of the hybrid models' prefill on the 5th-generation tensor cores:
// out[token, feature] = sum_k A[token, k] * W[feature, k], fp32 accumulation in tensor memory.
//
// Persistent, warp-specialised: one producer thread (TMA, 128-byte swizzle), one MMA thread
// (tcgen05.mma, M = 128 tokens, N = kBN features), four epilogue warps that read one of two
// accumulators back while the other is being filled.  The epilogue goes through shared memory so
// that stores are row segments: plus the bias, times the layer scale into the 32-bit residual stream,
// in bf16, or the gated unit of neighbouring columns in bf16.
#include "hybrid_kernels.h"
#include "hybrid_tcgen05.cuh"

namespace mkbh {
namespace {

constexpr int kBM = 128, kBK = 64;
constexpr int kGemmThreads = 192;
constexpr int kEpiStride = 33;  // floats per row of a warp's 32 x 32 transpose buffer

template <int kBN>
struct Geo {
    static constexpr int kStageBytes = (kBM + kBN) * kBK * 2;
    static constexpr int kStages = kBN == 256 ? 4 : kBN == 128 ? 6 : 8;
    static constexpr int kEpi = kStages * kStageBytes;
    static constexpr int kBars = kEpi + 4 * 32 * kEpiStride * 4;
    static constexpr int kNumBars = 2 * kStages + 4;
    static constexpr int kCtl = kBars + kNumBars * 8;
    static constexpr int kTotal = kCtl + 16;
    static constexpr int kAlloc = kTotal + 1024;
    static_assert(kAlloc <= 227 * 1024, "");
};

struct Shape {
    int T, N, K, tiles_m, tiles;
    unsigned long long timeout_ns;
    int* status;
};

template <int kBN>
__global__ void __launch_bounds__(kGemmThreads, 1)
gemm_bf16_kernel(const __grid_constant__ CUtensorMap amap, const __grid_constant__ CUtensorMap wmap, const Shape s,
                 const GemmEpilogue e) {
    using G = Geo<kBN>;
    extern __shared__ uint8_t raw[];
    const uint32_t raw32 = mkb::smem_u32(raw), base = (raw32 + 1023u) & ~1023u;
    uint8_t* gbase = raw + (base - raw32);
    volatile int* ctl = reinterpret_cast<volatile int*>(gbase + G::kCtl);  // [0] dead, [1] tensor-memory base
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    auto full = [&](int i) { return base + G::kBars + i * 8; };
    auto empty = [&](int i) { return base + G::kBars + (G::kStages + i) * 8; };
    auto acc_full = [&](int i) { return base + G::kBars + (2 * G::kStages + i) * 8; };
    auto acc_empty = [&](int i) { return base + G::kBars + (2 * G::kStages + 2 + i) * 8; };

    if (threadIdx.x == 0) {
        for (int i = 0; i < G::kStages; ++i) {
            mkb::mbar_init(full(i), 1);
            mkb::mbar_init(empty(i), 1);
        }
        for (int i = 0; i < 2; ++i) {
            mkb::mbar_init(acc_full(i), 1);
            mkb::mbar_init(acc_empty(i), 4);
        }
        ctl[0] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(base + G::kCtl + 4),
                     "r"((uint32_t)(2 * kBN))
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = (uint32_t)ctl[1];
    const int ksteps = (s.K + kBK - 1) / kBK;

    if (warp == 0 && lane == 0) {
        uint32_t it = 0;
        bool ok = true;
        for (int tile = blockIdx.x; tile < s.tiles && ok; tile += gridDim.x) {
            const int m0 = (tile % s.tiles_m) * kBM, n0 = (tile / s.tiles_m) * kBN;
            for (int k = 0; k < ksteps; ++k, ++it) {
                const int st = it % G::kStages;
                if (!tc_wait(empty(st), ((it / G::kStages) & 1u) ^ 1u, ctl, s.timeout_ns, s.status, 0)) {
                    ok = false;
                    break;
                }
                const uint32_t dst = base + st * G::kStageBytes;
                mkb::mbar_expect_tx(full(st), G::kStageBytes);
                tc_tma_2d(dst, &amap, k * kBK, m0, full(st));
                tc_tma_2d(dst + kBM * kBK * 2, &wmap, k * kBK, n0, full(st));
            }
        }
        // no copy may be in flight when the CTA's shared memory goes away
        for (uint32_t i = it > (uint32_t)G::kStages ? it - G::kStages : 0u; i < it; ++i)
            tc_wait(full(i % G::kStages), (i / G::kStages) & 1u, nullptr, s.timeout_ns, s.status, 0);
    } else if (warp == 1 && lane == 0) {
        const uint32_t idesc = tc_idesc(kBM, kBN);
        uint32_t it = 0, acc = 0;
        bool ok = true;
        for (int tile = blockIdx.x; tile < s.tiles && ok; tile += gridDim.x, ++acc) {
            const uint32_t buf = acc & 1u;
            ok = tc_wait(acc_empty(buf), ((acc >> 1) & 1u) ^ 1u, ctl, s.timeout_ns, s.status, 1);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            for (int k = 0; k < ksteps; ++k, ++it) {
                const int st = it % G::kStages;
                ok = tc_wait(full(st), (it / G::kStages) & 1u, ctl, s.timeout_ns, s.status, 1);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t a = base + st * G::kStageBytes, w = a + kBM * kBK * 2;
#pragma unroll
                for (int kk = 0; kk < kBK / 16; ++kk)
                    tc_mma(tmem + buf * kBN, tc_desc(a + kk * 32), tc_desc(w + kk * 32), idesc, (uint32_t)((k | kk) != 0));
                tc_commit(empty(st));
            }
            if (ok) tc_commit(acc_full(buf));
        }
    } else if (warp >= 2) {
        const int q = warp & 3;  // the quarter of tensor memory's lanes this warp may read
        float* tr = reinterpret_cast<float*>(gbase + G::kEpi) + (warp - 2) * 32 * kEpiStride;
        uint32_t acc = 0;
        for (int tile = blockIdx.x; tile < s.tiles; tile += gridDim.x, ++acc) {
            const int m0 = (tile % s.tiles_m) * kBM + q * 32, n0 = (tile / s.tiles_m) * kBN;
            const uint32_t buf = acc & 1u;
            const bool ok = tc_wait(acc_full(buf), (acc >> 1) & 1u, ctl, s.timeout_ns, s.status, 2);
            if (!__all_sync(0xffffffffu, ok)) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int rows = min(32, s.T - m0);
            for (int c0 = 0; c0 < kBN; c0 += 32) {
                if (n0 + c0 >= s.N || rows <= 0) break;  // uniform over the warp
                uint32_t r[32];
                tc_load32(tmem + ((uint32_t)(q * 32) << 16) + buf * kBN + c0, r);
#pragma unroll
                for (int j = 0; j < 32; ++j) tr[lane * kEpiStride + j] = __uint_as_float(r[j]);
                __syncwarp();
                if (e.what == Result::kCast) {  // two rows at a time, two columns per lane
                    const int col = 2 * (lane & 15), n = n0 + c0 + col;
                    bf16* o = static_cast<bf16*>(e.cast) + (size_t)m0 * e.ld + n;
                    for (int i = lane >> 4; i < rows; i += 2) {
                        const float *v = tr + i * kEpiStride + col;
                        if (n + 1 < s.N) *reinterpret_cast<uint32_t*>(o + (size_t)i * e.ld) = mkb::pack_bf16x2(v[0], v[1]);
                        else if (n < s.N) o[(size_t)i * e.ld] = __float2bfloat16_rn(v[0]);
                    }
                } else if (e.what == Result::kGlu) {  // 16 units of a row per half warp
                    const int col = 2 * (lane & 15), n = n0 + c0 + col;
                    bf16* o = static_cast<bf16*>(e.cast) + (size_t)m0 * e.ld + n / 2;
                    if (n < s.N)  // (N is even)
                        for (int i = lane >> 4; i < rows; i += 2) {
                            const float* v = tr + i * kEpiStride + col;
                            o[(size_t)i * e.ld] = __float2bfloat16_rn(clamped_glu(v[0], v[1], e.limit, e.alpha));
                        }
                }
                const int n = n0 + c0 + lane;
                if (n < s.N && e.what <= Result::kAdd) {
                    float* o = e.out + (size_t)m0 * e.ld + n;
                    if (e.what == Result::kAdd) {
                        const float f = e.scale ? __ldg(e.scale + n) : 1.f;
                        // (this tile is the only writer of these elements: one addition each, in L2)
                        for (int i = 0; i < rows; ++i)
                            asm volatile("red.global.add.f32 [%0], %1;" ::"l"(o + (size_t)i * e.ld), "f"(f * tr[i * kEpiStride + lane])
                                         : "memory");
                    } else {
                        const float b = e.bias ? __ldg(e.bias + n) : 0.f;
                        for (int i = 0; i < rows; ++i) o[(size_t)i * e.ld] = tr[i * kEpiStride + lane] + b;
                    }
                }
                __syncwarp();
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mkb::mbar_arrive(acc_empty(buf));
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((uint32_t)(2 * kBN)) : "memory");
}

template <int kBN>
cudaError_t launch(const bf16* A, int64_t lda, const bf16* W, int64_t ldw, Shape s, const GemmEpilogue& e, int sms,
                   cudaStream_t st) {
    using G = Geo<kBN>;
    static bool set[64] = {};
    int dev = 0;
    cudaError_t err = cudaGetDevice(&dev);
    if (err != cudaSuccess) return err;
    if (!set[dev & 63]) {
        err = cudaFuncSetAttribute(gemm_bf16_kernel<kBN>, cudaFuncAttributeMaxDynamicSharedMemorySize, G::kAlloc);
        if (err != cudaSuccess) return err;
        set[dev & 63] = true;
    }
    CUtensorMap amap, wmap;
    if ((err = tc_map(&amap, A, s.K, s.T, lda, kBK, kBM)) != cudaSuccess) return err;
    if ((err = tc_map(&wmap, W, s.K, s.N, ldw, kBK, kBN)) != cudaSuccess) return err;
    s.tiles_m = (s.T + kBM - 1) / kBM;
    s.tiles = s.tiles_m * ((s.N + kBN - 1) / kBN);
    gemm_bf16_kernel<kBN><<<s.tiles < sms ? s.tiles : sms, kGemmThreads, G::kAlloc, st>>>(amap, wmap, s, e);
    return cudaGetLastError();
}

}  // namespace

cudaError_t gemm_bf16(const bf16* A, int64_t lda, const bf16* W, int64_t ldw, int T, int N, int K, const GemmEpilogue& e,
                      int* status, cudaStream_t st) {
    static int sms = 0;
    if (sms == 0) {
        int dev = 0;
        cudaError_t err = cudaGetDevice(&dev);
        if (err == cudaSuccess) err = cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
        if (err != cudaSuccess) return err;
    }
    Shape s{T, N, K, 0, 0, 2000000000ull, status};
    // the tile width with the shortest estimated time: full waves of tiles, wide tiles being cheaper per column
    const int tm = (T + kBM - 1) / kBM;
    auto cost = [&](int bn, float per_tile) {
        const int tiles = tm * ((N + bn - 1) / bn);
        return ((tiles + sms - 1) / sms) * per_tile;
    };
    const float c256 = cost(256, 1.f), c128 = cost(128, 0.56f), c64 = cost(64, 0.36f);
    if (c256 <= c128 && c256 <= c64) return launch<256>(A, lda, W, ldw, s, e, sms, st);
    if (c128 <= c64) return launch<128>(A, lda, W, ldw, s, e, sms, st);
    return launch<64>(A, lda, W, ldw, s, e, sms, st);
}

}  // namespace mkbh
