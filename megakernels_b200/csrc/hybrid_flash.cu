// Prefill attention of the one-map mixers (rotary, latent) on the 5th-generation tensor cores: 128
// queries of one head x tiles of up to 128 keys.
//
// Warp roles: a TMA producer, an MMA thread, eight softmax warps; two threads share a query row, half of
// a tile's keys each.
//   scores   S = Q K^T in tensor memory, two buffers: the next tile's scores are computed while this
//            tile's are in the softmax;
//   weights  go back to tensor memory as bf16 and are the A operand of
//   output   O += P V, V as it lies in the cache (MN-major), accumulated in tensor memory.
// Scores, maxima, exponentials and sums are fp32.  O refers to a row maximum that is replaced only when
// it is exceeded by more than 2^8: then the row's softmax thread rescales O itself.  A sink is a key
// without a value that is there from the start.  Outputs of rotated values are turned back at the end.
// Keys may come in two pieces (a latent's expanded part per head, its rotated part for all heads).
// A tile never crosses the point where a ring of cache rows wraps.
#include "hybrid_kernels.h"
#include "hybrid_tcgen05.cuh"

namespace mkbh {
namespace {

// A slab is 128 rows of 64 bf16 columns.  Queries lie in whole slabs per head, zero beyond the head's
// size; what a slab of keys or values holds beyond it (a neighbour's entries) meets those zeros, or
// output columns that are not stored.
constexpr int kRows = 128, kTile = 128, kSlab = kTile * 128;
constexpr int kSoftWarps = 8, kHalf = kTile / 2;
constexpr int kFlashThreads = 64 + 32 * kSoftWarps;
constexpr int kP = 2 * kTile, kOut = kP + kTile;  // tensor-memory columns: scores, weights (two buffers), output
constexpr float kSlack = 8.f;

struct FlashShape {
    int n, pos0, heads, per, split_slabs, rest_slabs, v_slabs, stages;
    int key_x, value_x, value_x0, key_y, value_y;  // columns of a head, first value column; rows of a head
    int window, chunk, ring, vdim;
    float scale;
    const float *temp, *sink, *value_rope;
    bf16* out;
    int64_t ldo;
    unsigned long long timeout_ns;
    int* status;
};
struct FlashMaps {
    CUtensorMap q, k, k_rest, v;
};
struct FlashSmem {  // byte offsets
    int q, k, v, row, bars, ctl, total;
    __host__ __device__ FlashSmem(int slabs, int v_slabs, int stages) {
        q = 0;
        k = slabs * kSlab;
        v = k + stages * slabs * kSlab;
        row = v + stages * v_slabs * kSlab;  // what the two threads of a row tell each other: [parity][half][row]
        bars = row + 4 * kRows * 4;
        ctl = bars + (1 + 4 * stages + 6 + 4) * 8;
        total = ctl + 16;
    }
};
// Tiles of the keys that some query of a block sees.
struct Tiles {
    int lo, hi, ring;
    __device__ __forceinline__ int first_key(const FlashShape& s, int p) const { return s.chunk > 0 ? p - p % s.chunk : max(0, p - s.window + 1); }
    __device__ __forceinline__ Tiles(const FlashShape& s, int p0, int p1) : hi(p1), ring(s.ring) { lo = first_key(s, p0); }
    __device__ __forceinline__ int row(int j) const { return j % ring; }
    __device__ __forceinline__ int len(int j) const { return min(min(kTile, hi - j + 1), ring - row(j)); }
};

// kE: value columns, in whole slabs
template <int kE>
__global__ void __launch_bounds__(kFlashThreads, 1) flash_tc_kernel(const __grid_constant__ FlashMaps maps, const FlashShape s) {
    extern __shared__ uint8_t raw[];
    const uint32_t raw32 = mkb::smem_u32(raw), base = (raw32 + 1023u) & ~1023u;
    const int slabs = s.split_slabs + s.rest_slabs, S = s.stages;
    const FlashSmem sm(slabs, s.v_slabs, S);
    volatile int* ctl = reinterpret_cast<volatile int*>(raw + (base - raw32) + sm.ctl);  // [0] dead, [1] tensor-memory base
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t bars = base + sm.bars, q_full = bars;
    auto k_full = [&](int i) { return bars + (1 + i) * 8; };
    auto k_empty = [&](int i) { return bars + (1 + S + i) * 8; };
    auto v_full = [&](int i) { return bars + (1 + 2 * S + i) * 8; };
    auto v_empty = [&](int i) { return bars + (1 + 3 * S + i) * 8; };
    auto s_full = [&](int i) { return bars + (1 + 4 * S + i) * 8; };
    auto p_full = [&](int i) { return bars + (3 + 4 * S + i) * 8; };
    auto o_done = [&](int i) { return bars + (5 + 4 * S + i) * 8; };
    auto meeting = [&](int i) { return bars + (7 + 4 * S + i) * 8; };
    const int h = blockIdx.x, g = h / s.per, t0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * kRows;
    const int nq = min(kRows, s.n - t0), p0 = s.pos0 + t0, p1 = p0 + nq - 1;
    const Tiles tiles(s, p0, p1);
    auto wait = [&](uint32_t bar, uint32_t parity, int role) { return tc_wait(bar, parity & 1u, ctl, s.timeout_ns, s.status, role); };

    if (threadIdx.x == 0) {
        mkb::mbar_init(q_full, 1);
        for (int i = 0; i < S; ++i) {
            mkb::mbar_init(k_full(i), 1);
            mkb::mbar_init(k_empty(i), 1);
            mkb::mbar_init(v_full(i), 1);
            mkb::mbar_init(v_empty(i), 1);
        }
        for (int i = 0; i < 2; ++i) {
            mkb::mbar_init(s_full(i), 1);
            mkb::mbar_init(p_full(i), kSoftWarps);
            mkb::mbar_init(o_done(i), 1);
        }
        for (int i = 0; i < 4; ++i) mkb::mbar_init(meeting(i), 2);
        ctl[0] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(base + sm.ctl + 4), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_before_sync();
    __syncthreads();
    tc_after_sync();
    const uint32_t tmem = (uint32_t)ctl[1];

    if (warp == 0 && lane == 0) {
        mkb::mbar_expect_tx(q_full, slabs * kSlab);
        for (int i = 0; i < slabs; ++i) tc_tma_2d(base + sm.q + i * kSlab, &maps.q, (h * slabs + i) * 64, t0, q_full);
        int issued = 0;
        bool ok = true;
        for (int j = tiles.lo; j <= tiles.hi && ok; j += tiles.len(j), ++issued) {
            const int st = issued % S, row = tiles.row(j);
            const uint32_t parity = (uint32_t)(issued / S) ^ 1u;
            ok = wait(k_empty(st), parity, 0);
            if (!ok) break;
            mkb::mbar_expect_tx(k_full(st), slabs * kSlab);
            const uint32_t kd = base + sm.k + st * slabs * kSlab;
            for (int i = 0; i < slabs; ++i) {
                if (i < s.split_slabs) tc_tma_2d(kd + i * kSlab, &maps.k, g * s.key_x + i * 64, g * s.key_y + row, k_full(st));
                else tc_tma_2d(kd + i * kSlab, &maps.k_rest, (i - s.split_slabs) * 64, row, k_full(st));
            }
            ok = wait(v_empty(st), parity, 0);
            if (!ok) break;  // (the keys of this tile are waited for below)
            mkb::mbar_expect_tx(v_full(st), s.v_slabs * kSlab);
            for (int i = 0; i < s.v_slabs; ++i)
                tc_tma_2d(base + sm.v + (st * s.v_slabs + i) * kSlab, &maps.v, s.value_x0 + g * s.value_x + i * 64, g * s.value_y + row, v_full(st));
        }
        // no copy may be in flight when the CTA's shared memory goes away
        auto drain = [&](uint32_t bar, uint32_t parity) { tc_wait(bar, parity & 1u, nullptr, s.timeout_ns, s.status, 0); };
        drain(q_full, 0);
        if (ok) {
            for (int i = issued > S ? issued - S : 0; i < issued; ++i) {
                drain(k_full(i % S), (uint32_t)(i / S));
                drain(v_full(i % S), (uint32_t)(i / S));
            }
        } else {  // a bounded time for whatever was issued
            const unsigned long long end = mkb::globaltimer_ns() + 1000000ull;
            while (mkb::globaltimer_ns() < end) {
            }
        }
    } else if (warp == 1 && lane == 0) {
        const uint32_t s_desc = tc_idesc(kRows, kTile), o_desc = tc_idesc(kRows, kE, true);
        auto scores = [&](int t) {  // tile t
            const int st = t % S;
            if (!wait(k_full(st), (uint32_t)(t / S), 1)) return false;
            tc_after_sync();
            const uint32_t q = base + sm.q, k = base + sm.k + st * slabs * kSlab;
            for (int i = 0; i < slabs; ++i)
#pragma unroll
                for (int kk = 0; kk < 4; ++kk)
                    tc_mma(tmem + (t & 1) * kTile, tc_desc(q + i * kSlab + kk * 32), tc_desc(k + i * kSlab + kk * 32), s_desc, (uint32_t)((i | kk) != 0));
            tc_commit(k_empty(st));
            tc_commit(s_full(t & 1));
            return true;
        };
        int count = 0;
        for (int j = tiles.lo; j <= tiles.hi; j += tiles.len(j)) ++count;
        bool ok = wait(q_full, 0, 1);
        for (int t = 0; t < 2 && t < count && ok; ++t) ok = scores(t);
        for (int t = 0; t < count && ok; ++t) {
            const int st = t % S;
            ok = wait(p_full(t & 1), (uint32_t)(t >> 1), 1) && wait(v_full(st), (uint32_t)(t / S), 1);
            if (!ok) break;
            tc_after_sync();
            const uint32_t v = base + sm.v + st * s.v_slabs * kSlab;
#pragma unroll
            for (int kk = 0; kk < kTile / 16; ++kk)
                tc_mma_ts(tmem + kOut, tmem + kP + (t & 1) * (kTile / 2) + kk * 8, tc_desc_mn(v + kk * 2048, kSlab), o_desc, (uint32_t)((t | kk) != 0));
            tc_commit(v_empty(st));
            tc_commit(o_done(t & 1));
            if (t + 2 < count) ok = scores(t + 2);  // (tile t's scores have been read: its weights are there)
        }
    } else if (warp >= 2) {
        const int quarter = warp & 3, half = (warp - 2) >> 2, r = quarter * 32 + lane;  // (a warp may touch 32 lanes of tensor memory)
        float* const mine = reinterpret_cast<float*>(raw + (base - raw32) + sm.row) + half * kRows + r;
        float* const other = mine + (half ? -kRows : kRows);
        auto meet = [&](int n) {  // the two warps of these rows, for the n-th time
            tc_before_sync();
            __syncwarp();
            if (lane == 0) mkb::mbar_arrive(meeting(quarter));
            const bool met = __all_sync(0xffffffffu, wait(meeting(quarter), (uint32_t)n, 2));
            tc_after_sync();
            return met;
        };
        const uint32_t lanes = tmem + ((uint32_t)(quarter * 32) << 16);
        const float log2e = 1.4426950408889634f, scale = s.scale * (s.temp ? __ldg(s.temp + h) : 1.f) * log2e;
        const int pos = p0 + min(r, nq - 1), row_lo = tiles.first_key(s, pos);
        const int warp_p0 = p0 + quarter * 32, warp_last_lo = tiles.first_key(s, min(warp_p0 + 31, p1));
        float top = s.sink ? __ldg(s.sink + h) * log2e : -INFINITY, sum = s.sink && half == 0 ? 1.f : 0.f;
        bool ok = true;
        int t = 0;
        for (int j = tiles.lo; j <= tiles.hi; j += tiles.len(j), ++t) {
            const int len = tiles.len(j);
            ok = __all_sync(0xffffffffu, wait(s_full(t & 1), (uint32_t)(t >> 1), 2));
            if (!ok) break;
            tc_after_sync();
            const uint32_t at = lanes + (t & 1) * kTile;
            uint32_t x[kHalf];
#pragma unroll
            for (int c = 0; c < kHalf; c += 32) tc_load32_async(at + half * kHalf + c, x + c);
#pragma unroll
            for (int c = 0; c < kHalf; c += 32) tc_loaded32(x + c);
            const bool whole = len == kTile && j >= warp_last_lo && j + kTile - 1 <= warp_p0;  // every row sees the whole tile
            const float mul = whole ? scale : 1.f;
            float m4[4];
            if (whole && scale < 0.f) {  // the smallest product is the largest score
#pragma unroll
                for (int i = 0; i < 4; ++i) m4[i] = INFINITY;
#pragma unroll
                for (int i = 0; i < kHalf; ++i) m4[i & 3] = fminf(m4[i & 3], __uint_as_float(x[i]));
#pragma unroll
                for (int i = 0; i < 4; ++i) m4[i] *= scale;
            } else if (whole) {
#pragma unroll
                for (int i = 0; i < 4; ++i) m4[i] = -INFINITY;
#pragma unroll
                for (int i = 0; i < kHalf; ++i) m4[i & 3] = fmaxf(m4[i & 3], __uint_as_float(x[i]));
#pragma unroll
                for (int i = 0; i < 4; ++i) m4[i] *= scale;
            } else {
                const int first = row_lo - j - half * kHalf, last = min(pos - j, len - 1) - half * kHalf;
#pragma unroll
                for (int i = 0; i < 4; ++i) m4[i] = -INFINITY;
#pragma unroll
                for (int i = 0; i < kHalf; ++i) {
                    const float z = i >= first && i <= last ? __uint_as_float(x[i]) * scale : -INFINITY;
                    m4[i & 3] = fmaxf(m4[i & 3], z);
                    x[i] = __float_as_uint(z);
                }
            }
            const int parity = (t & 1) * 2 * kRows;
            mine[parity] = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
            ok = meet(t);
            if (!ok) break;
            const float best = fmaxf(mine[parity], other[parity]);
            const bool raise = best > top + kSlack;
            if (__any_sync(0xffffffffu, raise)) {
                const float f = raise ? exp2f(top - best) : 1.f;  // (0 from minus infinity)
                if (raise) top = best;
                sum *= f;
                if (t > 0) {
                    ok = __all_sync(0xffffffffu, wait(o_done((t - 1) & 1), (uint32_t)((t - 1) >> 1), 2));
                    if (!ok) break;
                    tc_after_sync();
#pragma unroll 1
                    for (int c = half * kE / 2; c < (half + 1) * kE / 2; c += 32) {
                        uint32_t o[32];
                        tc_load32(lanes + kOut + c, o);
#pragma unroll
                        for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
                        tc_store16(lanes + kOut + c, o);
                        tc_store16(lanes + kOut + c + 16, o + 16);
                    }
                }
            }
            if (t > 1) {  // the weights of two tiles before have been read
                ok = __all_sync(0xffffffffu, wait(o_done(t & 1), (uint32_t)((t - 2) >> 1), 2));
                if (!ok) break;
                tc_after_sync();
            }
            const float off = top == -INFINITY ? 0.f : top;
            float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int c = 0; c < kHalf; c += 16) {
                uint32_t w[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    float z[2];
#pragma unroll
                    for (int k = 0; k < 2; ++k)
                        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(z[k]) : "f"(fmaf(__uint_as_float(x[c + 2 * i + k]), mul, -off)));
                    part[i & 3] += z[0] + z[1];
                    w[i] = mkb::pack_bf16x2(z[0], z[1]);
                }
                tc_store8(lanes + kP + (t & 1) * (kTile / 2) + (half * kHalf + c) / 2, w);
            }
            sum += (part[0] + part[1]) + (part[2] + part[3]);
            tc_stored();
            tc_before_sync();
            __syncwarp();
            if (lane == 0) mkb::mbar_arrive(p_full(t & 1));
        }
        if (ok) ok = __all_sync(0xffffffffu, wait(o_done((t - 1) & 1), (uint32_t)((t - 1) >> 1), 2));
        if (ok) {
            tc_after_sync();
            const int parity = (t & 1) * 2 * kRows;
            mine[parity] = sum;
            ok = meet(t);
            if (ok) sum += other[parity];
            const float inv = sum > 0.f ? 1.f / sum : 0.f;
            const float2* turn = s.value_rope ? reinterpret_cast<const float2*>(s.value_rope) + (size_t)pos * (s.vdim / 2) : nullptr;
            bf16* dst = s.out + (size_t)(t0 + r) * s.ldo + h * s.vdim;
#pragma unroll 1
            for (int c = half * kE / 2; c < (half + 1) * kE / 2; c += 32) {
                uint32_t o[32];
                tc_load32(lanes + kOut + c, o);
                if (r >= nq) continue;
#pragma unroll
                for (int e = 0; e < 32; e += 8) {
                    if (c + e >= s.vdim) break;  // (a multiple of 8)
                    uint32_t w[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        float a = __uint_as_float(o[e + 2 * i]) * inv, b = __uint_as_float(o[e + 2 * i + 1]) * inv;
                        if (turn != nullptr) {
                            const float2 z = __ldg(turn + (c + e) / 2 + i);
                            const float y = a * z.x + b * z.y;
                            b = b * z.x - a * z.y;
                            a = y;
                        }
                        w[i] = mkb::pack_bf16x2(a, b);
                    }
                    *reinterpret_cast<uint4*>(dst + c + e) = make_uint4(w[0], w[1], w[2], w[3]);
                }
            }
        }
    }
    tc_before_sync();
    __syncthreads();
    if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
}

int slabs_of(int n) { return (n + 63) / 64; }
constexpr int kLimit = 227 * 1024 - 1024;
int stages_for(int slabs, int v_slabs) {
    for (int st = 4; st >= 2; --st)
        if (FlashSmem(slabs, v_slabs, st).total <= kLimit) return st;
    return 0;
}

template <int kE>
cudaError_t launch(const FlashMaps& maps, const FlashShape& s, cudaStream_t stream) {
    static bool set[64] = {};
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    if (!set[dev & 63]) {
        e = cudaFuncSetAttribute(flash_tc_kernel<kE>, cudaFuncAttributeMaxDynamicSharedMemorySize, kLimit + 1024);
        if (e != cudaSuccess) return e;
        set[dev & 63] = true;
    }
    const int bytes = FlashSmem(s.split_slabs + s.rest_slabs, s.v_slabs, s.stages).total + 1024;
    flash_tc_kernel<kE><<<dim3(s.heads, (s.n + kRows - 1) / kRows), kFlashThreads, bytes, stream>>>(maps, s);
    return cudaGetLastError();
}

}  // namespace

bool flash_tc_supported(const MkbhLayer& L) {
    const int rest = L.mixer == MKBH_LATENT_ATTENTION ? L.rot_dim : 0;
    return L.dim % 8 == 0 && rest % 8 == 0 && L.vdim % 8 == 0 && L.vdim <= 128 && L.cache_keep == 0 && L.keep_first == 0 &&
           stages_for(slabs_of(L.dim) + slabs_of(rest), slabs_of(L.vdim)) >= 2;
}

cudaError_t flash_tc(const MkbhGlobals& g, const MkbhLayer& L, bf16* out, int64_t ldo, cudaStream_t stream) {
    const KeySource<bf16> src = key_source<bf16>(g, L);
    const int A = src.split, B = src.rest, H = L.heads, G = H / src.per, rows = L.cache_ring;
    const bool latent = L.mixer == MKBH_LATENT_ATTENTION;
    const int slabs = query_head<bf16>(L) / 64;
    FlashMaps m;
    cudaError_t e;
    if ((e = tc_map(&m.q, static_cast<const bf16*>(g.query), H * slabs * 64, g.num_tokens, H * slabs * 64, 64, kRows)) != cudaSuccess) return e;
    // (latent: all heads side by side, keys then values; rotary: one head's rows after the other's)
    const int columns = H * (L.dim + L.vdim);
    if ((e = tc_map(&m.k, src.keys, latent ? columns : A, latent ? rows : G * rows, src.key_ld, 64, kTile)) != cudaSuccess) return e;
    if ((e = tc_map(&m.v, latent ? src.keys : src.values, latent ? columns : L.vdim, latent ? rows : G * rows, src.value_ld, 64, kTile)) != cudaSuccess)
        return e;
    m.k_rest = m.k;
    if (B > 0 && (e = tc_map(&m.k_rest, src.shared, B, rows, src.shared_ld, 64, kTile)) != cudaSuccess) return e;
    FlashShape s{g.num_tokens, g.pos0, H, src.per, slabs_of(A), B > 0 ? slabs_of(B) : 0, slabs_of(L.vdim), 0,
                 latent ? A : 0, latent ? L.vdim : 0, latent ? H * A : 0, latent ? 0 : rows, latent ? 0 : rows,
                 L.window, L.chunk, rows, L.vdim, L.scale, L.temp, L.sink, L.value_rope, out, ldo, 2000000000ull, g.status};
    s.stages = stages_for(s.split_slabs + s.rest_slabs, s.v_slabs);
    return s.v_slabs == 1 ? launch<64>(m, s, stream) : launch<128>(m, s, stream);
}

}  // namespace mkbh
