// bf16 matrix product of the hybrid models' prefill on the 5th-generation tensor cores:
// out[token, feature] = sum_k A[token, k] * W[feature, k], fp32 accumulation in tensor memory.
//
// Persistent, warp-specialised: one producer thread (TMA, 128-byte swizzle), one MMA thread
// (tcgen05.mma, M = 128 tokens, N = kBN features), four epilogue warps that read one of two
// accumulators back while the other is being filled.  The epilogue goes through shared memory so
// that stores are row segments: plus the bias, times the layer scale into the 32-bit residual stream,
// in bf16, or the gated unit of neighbouring columns in bf16.
#include "hybrid_kernels.h"

#include <cuda.h>

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

// Bounded wait; on expiry records the fault, marks the CTA as dead and returns false.
__device__ __noinline__ bool wait_slow(uint32_t bar, uint32_t parity, volatile int* dead, const Shape& s, int role) {
    const unsigned long long t0 = mkb::globaltimer_ns();
    for (uint32_t spins = 1;; ++spins) {
        if (mkb::mbar_try_wait(bar, parity)) return true;
        if ((spins & 63u) == 0) {
            if (dead != nullptr && *dead) return false;
            if (mkb::globaltimer_ns() - t0 > s.timeout_ns) {
                if (s.status != nullptr && atomicCAS(&s.status[0], 0, (int)MKBH_ERR_DEVICE_TIMEOUT) == 0) {
                    s.status[1] = blockIdx.x;
                    s.status[2] = -1;
                    s.status[3] = -1;
                    s.status[4] = role;
                }
                if (dead != nullptr) *dead = 1;
                return false;
            }
        }
    }
}
__device__ __forceinline__ bool wait_bar(uint32_t bar, uint32_t parity, volatile int* dead, const Shape& s, int role) {
    if (mkb::mbar_try_wait(bar, parity)) return true;
    return wait_slow(bar, parity, dead, s, role);
}

__device__ __forceinline__ void tma_2d(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(
            dst),
        "l"(map), "r"(x), "r"(y), "r"(bar)
        : "memory");
}
// K-major operand tile with the 128-byte swizzle: rows 128 bytes apart, groups of 8 rows 1024 bytes apart
__device__ __forceinline__ uint64_t smem_desc(uint32_t addr) {
    return (uint64_t)((addr & 0x3FFFFu) >> 4) | ((uint64_t)1 << 16) | ((uint64_t)(1024 >> 4) << 32) |
           ((uint64_t)1 << 46) | ((uint64_t)2 << 61);
}
__device__ __forceinline__ void mma_f16(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.u32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(d),
        "l"(a), "l"(b), "r"(idesc), "r"(accumulate)
        : "memory");
}
__device__ __forceinline__ void commit(uint32_t bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void tmem_ld32(uint32_t addr, uint32_t (&r)[32]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,"
        "%30,%31}, [%32];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
          "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
          "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
          "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
        : "r"(addr));
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}

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
                if (!wait_bar(empty(st), ((it / G::kStages) & 1u) ^ 1u, ctl, s, 0)) {
                    ok = false;
                    break;
                }
                const uint32_t dst = base + st * G::kStageBytes;
                mkb::mbar_expect_tx(full(st), G::kStageBytes);
                tma_2d(dst, &amap, k * kBK, m0, full(st));
                tma_2d(dst + kBM * kBK * 2, &wmap, k * kBK, n0, full(st));
            }
        }
        // no copy may be in flight when the CTA's shared memory goes away
        for (uint32_t i = it > (uint32_t)G::kStages ? it - G::kStages : 0u; i < it; ++i)
            wait_bar(full(i % G::kStages), (i / G::kStages) & 1u, nullptr, s, 0);
    } else if (warp == 1 && lane == 0) {
        const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kBN >> 3) << 17) | ((uint32_t)(kBM >> 4) << 24);
        uint32_t it = 0, acc = 0;
        bool ok = true;
        for (int tile = blockIdx.x; tile < s.tiles && ok; tile += gridDim.x, ++acc) {
            const uint32_t buf = acc & 1u;
            ok = wait_bar(acc_empty(buf), ((acc >> 1) & 1u) ^ 1u, ctl, s, 1);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            for (int k = 0; k < ksteps; ++k, ++it) {
                const int st = it % G::kStages;
                ok = wait_bar(full(st), (it / G::kStages) & 1u, ctl, s, 1);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t a = base + st * G::kStageBytes, w = a + kBM * kBK * 2;
#pragma unroll
                for (int kk = 0; kk < kBK / 16; ++kk)
                    mma_f16(tmem + buf * kBN, smem_desc(a + kk * 32), smem_desc(w + kk * 32), idesc, (uint32_t)((k | kk) != 0));
                commit(empty(st));
            }
            if (ok) commit(acc_full(buf));
        }
    } else if (warp >= 2) {
        const int q = warp & 3;  // the quarter of tensor memory's lanes this warp may read
        float* tr = reinterpret_cast<float*>(gbase + G::kEpi) + (warp - 2) * 32 * kEpiStride;
        uint32_t acc = 0;
        for (int tile = blockIdx.x; tile < s.tiles; tile += gridDim.x, ++acc) {
            const int m0 = (tile % s.tiles_m) * kBM + q * 32, n0 = (tile / s.tiles_m) * kBN;
            const uint32_t buf = acc & 1u;
            const bool ok = wait_bar(acc_full(buf), (acc >> 1) & 1u, ctl, s, 2);
            if (!__all_sync(0xffffffffu, ok)) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int rows = min(32, s.T - m0);
            for (int c0 = 0; c0 < kBN; c0 += 32) {
                if (n0 + c0 >= s.N || rows <= 0) break;  // uniform over the warp
                uint32_t r[32];
                tmem_ld32(tmem + ((uint32_t)(q * 32) << 16) + buf * kBN + c0, r);
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

typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                             const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                             CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

cudaError_t operand_map(CUtensorMap* map, const bf16* ptr, int K, int rows, int64_t ld, int box_rows) {
    static EncodeFn encode = nullptr;
    if (encode == nullptr) {
        void* fn = nullptr;
        cudaDriverEntryPointQueryResult q;
        cudaError_t e = cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &q);
        if (e != cudaSuccess) return e;
        if (q != cudaDriverEntryPointSuccess || fn == nullptr) return cudaErrorNotSupported;
        encode = reinterpret_cast<EncodeFn>(fn);
    }
    const cuuint64_t dims[2] = {(cuuint64_t)K, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {kBK, (cuuint32_t)box_rows}, elem[2] = {1, 1};
    const CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<bf16*>(ptr), dims, strides, box, elem,
                              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? cudaSuccess : cudaErrorInvalidValue;
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
    if ((err = operand_map(&amap, A, s.K, s.T, lda, kBM)) != cudaSuccess) return err;
    if ((err = operand_map(&wmap, W, s.K, s.N, ldw, kBN)) != cudaSuccess) return err;
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
