// Decode megakernel of the hybrid models: one token of one sequence in one persistent launch.
//
// The scheme of megakernel.cu - one CTA per SM, an instruction queue per CTA, a ring of weight
// stages in shared memory that a loader thread keeps full across instruction boundaries, counters
// in HBM that order the phases - for layers that are listed one by one (delta-rule recurrence or
// windowed differential attention, optional PolyNorm feed-forward) and for any sizes:
//   * a weight block is a run of whole rows, contiguous in memory, so a stage is ONE untiled bulk
//     copy (no tensor maps, no divisibility rules beyond the zero padding of a row to 16 bytes);
//   * 16 consumer warps multiply from shared memory with fp32 FMA (batch 1 is bandwidth-bound), the
//     same code for bf16 and float weights; every warp owns a fixed slice of the input columns, whose
//     activations stay in registers for the whole instruction;
//   * every output row has exactly one owner, which also adds it to the 32-bit residual stream: no
//     atomics on data, bit-identical results from run to run;
//   * whatever does not depend on the token (recurrent state, older keys and values, low-rank decay
//     factors) is fetched before an instruction waits for its producers;
//   * every wait is bounded and reports into the status record.
#include "hybrid_kernels.h"

#include <cstring>

namespace mkbh {
namespace {

using mkb::globaltimer_ns;
using mkb::ld_acquire_gpu;
using mkb::ld_cg_f32;
using mkb::lds_v4;
using mkb::mbar_arrive;
using mkb::mbar_expect_tx;
using mkb::mbar_init;
using mkb::mbar_try_wait;
using mkb::red_release_gpu_add;
using mkb::smem_u32;

constexpr int kConsumerWarps = 16;
constexpr int kConsumers = kConsumerWarps * 32;
constexpr int kBlock = kConsumers + 32;
constexpr int kStage = 32768;
constexpr int kMaxStages = 6;
constexpr int kPartFloats = 4096;      // per-row, per-column-group partial sums of an instruction
constexpr int kScratchMin = 40 * 1024; // activation / mixer scratch, at least
constexpr int kSmemLimit = 226 * 1024;
constexpr int kMaxStateRows = 16;      // key channels of one column a thread carries (DELTA_STEP)
constexpr int kMaxAcc = 16;            // outputs a thread carries (ATTENTION)

struct Params {
    MkbhGlobals g;
    int stages, act_bytes;
    int attn_chunk;        // keys staged at a time
    int l2_window;         // stages the loader may prefetch into L2 beyond the ring
    unsigned long long timeout_ns;
};

struct Smem {  // byte offsets from the 128-byte aligned base
    int act, part, red, bars, ctl, total;
    __host__ __device__ Smem(int stages, int act_bytes) {
        act = stages * kStage;
        part = act + act_bytes;
        red = part + kPartFloats * 4;
        bars = red + 128 * 4;
        ctl = bars + 2 * kMaxStages * 8;
        total = ctl + 16 * 4;
    }
};

struct Ctx {
    const Params* p;
    const MkbhGlobals* g;
    uint32_t base;       // shared-window address
    float *act, *part, *red;
    uint32_t bars;
    volatile int* ctl;   // [0] CTA abort, [1] last-arriver verdict, [2] agreed abort
    int instr, opcode, pos;
    uint32_t slot, phase;  // consumer view of the ring
    __device__ uint32_t full(int s) const { return bars + s * 8; }
    __device__ uint32_t empty(int s) const { return bars + (kMaxStages + s) * 8; }
};

__device__ __forceinline__ void csync() { asm volatile("bar.sync 1, %0;" ::"n"(kConsumers) : "memory"); }

__device__ __forceinline__ void rec(const Ctx& c, int slot) {
    if (c.g->timings != nullptr && threadIdx.x == 0)
        c.g->timings[((size_t)blockIdx.x * c.g->queue_len + c.instr) * MKBH_TIMING_SLOTS + slot] =
            (int)(uint32_t)globaltimer_ns();
}

__device__ __noinline__ void report(const Ctx& c, int code, int role, int d0, int d1, int d2) {
    int* st = c.g->status;
    if (atomicCAS(&st[0], 0, code) == 0) {
        st[1] = blockIdx.x;
        st[2] = c.instr;
        st[3] = c.opcode;
        st[4] = role;
        st[5] = d0;
        st[6] = d1;
        st[7] = d2;
        __threadfence();
    }
    atomicExch(&st[15], 1);
    c.ctl[0] = 1;
}
__device__ __forceinline__ bool global_abort(const Ctx& c) {
    return *reinterpret_cast<volatile int*>(&c.g->status[15]) != 0;
}

__device__ __noinline__ bool bar_wait_slow(const Ctx& c, uint32_t bar, uint32_t parity, int role, bool honour_abort) {
    const unsigned long long t0 = globaltimer_ns();
    for (uint32_t spins = 1;; ++spins) {
        if (mbar_try_wait(bar, parity)) return true;
        if ((spins & 63u) == 0) {
            if (honour_abort && c.ctl[0]) return false;
            if (globaltimer_ns() - t0 > c.p->timeout_ns) {
                report(c, MKBH_ERR_DEVICE_TIMEOUT, role, -1, 0, 0);
                return false;
            }
        }
    }
}

__device__ __forceinline__ int* counter(const Ctx& c, int layer, int op) {
    return c.g->counters + 2 + layer * MKBH_BARRIERS_PER_LAYER + op;
}
__device__ __forceinline__ int threshold(const Ctx& c, int layer, int op) {
    return __ldg(c.g->arrivals + layer * MKBH_BARRIERS_PER_LAYER + op);
}

// One consumer thread's view of the abort word for all of them (the loader may set it at any time):
// true if they go on together.
__device__ __forceinline__ bool agree(const Ctx& c) {
    if (threadIdx.x == 0) c.ctl[2] = c.ctl[0];
    csync();
    return c.ctl[2] == 0;
}

// All consumers: wait until phase `op` of `layer` is complete.  false (uniformly): aborting.
__device__ bool wait_phase(const Ctx& c, int layer, int op) {
    if (threadIdx.x == 0) {
        const int* addr = counter(c, layer, op);
        const int thr = threshold(c, layer, op);
        unsigned long long t0 = 0;
        uint32_t spins = 0;
        while (ld_acquire_gpu(addr) < thr) {
            if ((++spins & 63u) == 0) {
                if (c.ctl[0]) break;
                if (global_abort(c)) {
                    c.ctl[0] = 1;
                    break;
                }
                const unsigned long long now = globaltimer_ns();
                if (t0 == 0) t0 = now;
                else if (now - t0 > c.p->timeout_ns) {
                    report(c, MKBH_ERR_DEVICE_TIMEOUT, 1, layer, op, ld_acquire_gpu(addr));
                    break;
                }
            }
        }
    }
    return agree(c);
}
// All consumers, after their global writes: announce one arrival.
__device__ __forceinline__ void signal_phase(const Ctx& c, int layer, int op) {
    csync();
    if (threadIdx.x == 0) red_release_gpu_add(counter(c, layer, op), 1);
}
// Phase that completes the residual stream a layer reads.
__device__ __forceinline__ int last_phase(const MkbhLayer& L) { return L.ff ? MKBH_OP_DOWN : MKBH_OP_OUT_PROJ; }

// ---- the weight stream ------------------------------------------------------------------- //
struct Block {  // rows [r0, r1) of a matrix of `row_bytes` rows
    const uint8_t* w;
    int r0, r1, row_bytes;
};
template <typename T>
__device__ __forceinline__ bool weight_block(const MkbhGlobals& g, const int* w, Block& b) {
    const int op = __ldg(w), layer = __ldg(w + 1);
    const MkbhLayer* L = g.layers_device + layer;
    int K;
    switch (op) {
        case MKBH_OP_NORM_PROJ: b.w = (const uint8_t*)L->in_w; K = g.width; break;
        case MKBH_OP_OUT_PROJ:
            b.w = (const uint8_t*)L->out_w;
            K = L->heads * (L->mixer == MKBH_DELTA_RULE ? L->dim : L->vdim);
            break;
        case MKBH_OP_NORM_UP: b.w = (const uint8_t*)L->up_w; K = g.width; break;
        case MKBH_OP_DOWN: b.w = (const uint8_t*)L->down_w; K = L->ff; break;
        case MKBH_OP_HEAD: b.w = (const uint8_t*)g.head; K = g.width; break;
        default: return false;
    }
    b.r0 = __ldg(w + 2);
    b.r1 = __ldg(w + 3);
    b.row_bytes = pad8(K) * (int)sizeof(T);
    return true;
}

template <typename T>
struct Cursor {  // the queue's weight blocks as a flat sequence of stages
    int i = 0, row = 0;
    bool open = false;
    Block b;
    __device__ bool next(const MkbhGlobals& g, const int* queue, const uint8_t*& src, uint32_t& bytes) {
        while (!open) {
            if (i >= g.queue_len) return false;
            if (weight_block<T>(g, queue + (size_t)i * MKBH_INTS_PER_INSTRUCTION, b) && b.r1 > b.r0) {
                open = true;
                row = b.r0;
            } else {
                ++i;
            }
        }
        const int n = min(kStage / b.row_bytes, b.r1 - row);
        src = b.w + (size_t)row * b.row_bytes;
        bytes = (uint32_t)(n * b.row_bytes);
        row += n;
        if (row >= b.r1) {
            open = false;
            ++i;
        }
        return true;
    }
};

template <typename T>
__device__ void loader_main(Ctx& c) {
    const MkbhGlobals& g = *c.g;
    const int* queue = g.instructions + (size_t)blockIdx.x * g.queue_len * MKBH_INTS_PER_INSTRUCTION;
    const uint64_t policy = mkb::l2_policy_evict_first();
    Cursor<T> cur, pre;
    uint32_t issued = 0, ahead = 0;  // stages copied, stages prefetched or copied
    const uint8_t* src;
    uint32_t bytes;
    bool more = true;
    const int S = c.p->stages;
    while (cur.next(g, queue, src, bytes)) {
        const int slot = issued % S;
        const uint32_t parity = ((issued / S) & 1u) ^ 1u;
        if (ahead <= issued && more) {  // keep the look-ahead cursor in front of the ring
            const uint8_t* s2;
            uint32_t b2;
            more = pre.next(g, queue, s2, b2);
            ++ahead;
        }
        while (!mbar_try_wait(c.empty(slot), parity)) {
            if (more && ahead < issued + (uint32_t)c.p->l2_window) {
                const uint8_t* s2;
                uint32_t b2;
                more = pre.next(g, queue, s2, b2);
                if (more)
                    asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(s2), "r"(b2) : "memory");
                ++ahead;
                continue;
            }
            if (!bar_wait_slow(c, c.empty(slot), parity, 0, true)) goto drain;
            break;
        }
        mbar_expect_tx(c.full(slot), bytes);
        mkb::tma_bulk_g2s(c.base + slot * kStage, src, bytes, c.full(slot), policy);
        ++issued;
    }
drain:  // no copy may be in flight when the CTA's shared memory goes away
    for (uint32_t s = issued > (uint32_t)S ? issued - S : 0u; s < issued; ++s)
        if (!mbar_try_wait(c.full(s % S), (s / S) & 1u)) bar_wait_slow(c, c.full(s % S), (s / S) & 1u, 0, false);
}

// ---- matrix-vector products ---------------------------------------------------------------- //
template <typename T> struct Chunk;  // 16 bytes of weights times the matching activations
template <> struct Chunk<float> {
    static constexpr int kElems = 4;
    __device__ static __forceinline__ float dot(const uint4& w, const float* a, float acc) {
        acc = fmaf(__uint_as_float(w.x), a[0], acc);
        acc = fmaf(__uint_as_float(w.y), a[1], acc);
        acc = fmaf(__uint_as_float(w.z), a[2], acc);
        return fmaf(__uint_as_float(w.w), a[3], acc);
    }
};
template <> struct Chunk<bf16> {
    static constexpr int kElems = 8;
    __device__ static __forceinline__ float dot(const uint4& w, const float* a, float acc) {
        const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            acc = fmaf(mkb::bf16_lo(u[i]), a[2 * i], acc);
            acc = fmaf(mkb::bf16_hi(u[i]), a[2 * i + 1], acc);
        }
        return acc;
    }
};

// Column groups of an input of `chunks` 16-byte chunks: warps that share a row.
__host__ __device__ inline int column_groups(int chunks) {
    int n = 1;
    while (n < kConsumerWarps && n * 32 < chunks) n *= 2;
    return n;
}

// Multiply the instruction's rows with the activations in c.act; partial sums [row][group] to
// c.part.  Ends with a consumer barrier.  false (uniformly): aborting.
template <typename T, int kPer>
__device__ __noinline__ bool matvec_rows(Ctx& c, const Block& b, int groups) {
    constexpr int E = Chunk<T>::kElems;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int cg = warp & (groups - 1), rg = warp / groups, nrg = kConsumerWarps / groups;
    const int chunks = b.row_bytes / 16;
    float a[kPer * E];
    uint32_t off[kPer];
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const int ch = (k * groups + cg) * 32 + lane;
        off[k] = ch < chunks ? (uint32_t)ch * 16u : 0u;
#pragma unroll
        for (int e = 0; e < E; ++e) a[k * E + e] = ch < chunks ? c.act[ch * E + e] : 0.f;
    }
    const int per_stage = kStage / b.row_bytes;
    uint32_t slot = c.slot, phase = c.phase;
    bool ok = true;
    for (int r0 = b.r0; r0 < b.r1; r0 += per_stage) {
        const int n = min(per_stage, b.r1 - r0);
        bool mine = mbar_try_wait(c.full(slot), phase) || bar_wait_slow(c, c.full(slot), phase, 1, true);
        if (!__all_sync(0xffffffffu, mine)) {
            ok = false;
            break;
        }
        const uint32_t stage = c.base + slot * kStage;
        for (int r = rg; r < n; r += 4 * nrg) {
            float v[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int row = r + j * nrg;
                v[j] = 0.f;
                if (row < n) {  // uniform over the warp
                    const uint32_t addr = stage + (uint32_t)row * (uint32_t)b.row_bytes;
#pragma unroll
                    for (int k = 0; k < kPer; ++k) v[j] = Chunk<T>::dot(lds_v4(addr + off[k]), a + k * E, v[j]);
                }
            }
            // four sums over 32 lanes in six shuffles: lane quarter q ends up with row q
            const bool up = lane & 16, up2 = lane & 8;
            float x0 = up ? v[2] : v[0], x1 = up ? v[3] : v[1];
            x0 += __shfl_xor_sync(0xffffffffu, up ? v[0] : v[2], 16);
            x1 += __shfl_xor_sync(0xffffffffu, up ? v[1] : v[3], 16);
            float y = up2 ? x1 : x0;
            y += __shfl_xor_sync(0xffffffffu, up2 ? x0 : x1, 8);
            y += __shfl_xor_sync(0xffffffffu, y, 4);
            y += __shfl_xor_sync(0xffffffffu, y, 2);
            y += __shfl_xor_sync(0xffffffffu, y, 1);
            const int row = r + (lane >> 3) * nrg;
            if ((lane & 7) == 0 && row < n) c.part[(r0 - b.r0 + row) * groups + cg] = y;
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(c.empty(slot));
        if (++slot == (uint32_t)c.p->stages) {
            slot = 0;
            phase ^= 1u;
        }
    }
    c.slot = slot;
    c.phase = phase;
    if (!ok) c.ctl[0] = 1;
    csync();
    return agree(c);
}

template <typename T>
__device__ __forceinline__ bool matvec(Ctx& c, const Block& b, int& groups) {
    const int chunks = b.row_bytes / 16;
    groups = column_groups(chunks);
    if (chunks <= groups * 32) return matvec_rows<T, 1>(c, b, groups);
    if (chunks <= groups * 64) return matvec_rows<T, 2>(c, b, groups);
    return matvec_rows<T, 4>(c, b, groups);
}
__device__ __forceinline__ float row_sum(const Ctx& c, int i, int groups) {
    float s = 0.f;
    for (int k = 0; k < groups; ++k) s += c.part[i * groups + k];
    return s;
}

template <int N>
__device__ __forceinline__ void csum(const Ctx& c, float (&v)[N]) {  // totals over the consumers
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
    for (int n = 0; n < N; ++n) {
        v[n] = warp_sum(v[n]);
        if (lane == 0) c.red[n * kConsumerWarps + warp] = v[n];
    }
    csync();
#pragma unroll
    for (int n = 0; n < N; ++n) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < kConsumerWarps; ++w) s += c.red[n * kConsumerWarps + w];
        v[n] = s;
    }
    csync();
}

// ---- activations ------------------------------------------------------------------------- //
// Layer norm of the residual stream (or of the token's embedding, which `publish` also writes out).
template <typename T>
__device__ __noinline__ void norm_activation(const Ctx& c, const float* w, bool embedding, bool publish) {
    const MkbhGlobals& g = *c.g;
    const int K = g.width, tid = threadIdx.x;
    float s[1] = {0.f};
    if (embedding) {
        int tok = __ldg(g.tokens);
        tok = tok < 0 ? 0 : tok >= g.vocab ? g.vocab - 1 : tok;
        const T* e = static_cast<const T*>(g.embed) + (size_t)tok * K;
        const T* q = static_cast<const T*>(g.pos) + (size_t)c.pos * K;
        for (int i = tid; i < K; i += kConsumers) {
            const float x = to_f(e[i]) * g.embed_scale + to_f(q[i]);
            c.act[i] = x;
            if (publish) g.x[i] = x;
            s[0] += x;
        }
    } else {
#pragma unroll 4
        for (int i = tid; i < K; i += kConsumers) {
            const float x = ld_cg_f32(g.x + i);
            c.act[i] = x;
            s[0] += x;
        }
    }
    csum<1>(c, s);
    const float mean = s[0] / K;
    s[0] = 0.f;
    for (int i = tid; i < K; i += kConsumers) {
        const float d = c.act[i] - mean;
        s[0] += d * d;
    }
    csum<1>(c, s);
    const float inv = 1.f / sqrtf(s[0] / K + g.eps);
    for (int i = tid; i < K; i += kConsumers) c.act[i] = (c.act[i] - mean) * inv * __ldg(w + i);
    for (int i = K + tid; i < pad8(K); i += kConsumers) c.act[i] = 0.f;
    csync();
}

// Mixer output as the output projection reads it.
__device__ __noinline__ void mixed_activation(const Ctx& c, const MkbhLayer& L) {
    const MkbhGlobals& g = *c.g;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    int K;
    if (L.mixer == MKBH_DELTA_RULE) {
        K = L.heads * L.dim;
        for (int h = warp; h < L.heads; h += kConsumerWarps) {
            float s = 0.f;
            for (int i = lane; i < L.dim; i += 32) {
                const float o = ld_cg_f32(g.mixed + h * L.dim + i);
                c.act[h * L.dim + i] = o;
                s += o * o;
            }
            const float inv = 1.f / sqrtf(warp_sum(s) / L.dim + g.eps);
            for (int i = lane; i < L.dim; i += 32) {
                const int j = h * L.dim + i;
                c.act[j] *= inv * __ldg(L.out_norm + j) * sigmoid_f(ld_cg_f32(g.proj + 4 * K + j));
            }
        }
    } else {
        K = L.heads * L.vdim;
        for (int i = tid; i < K; i += kConsumers) c.act[i] = ld_cg_f32(g.mixed + i);
    }
    for (int i = K + tid; i < pad8(K); i += kConsumers) c.act[i] = 0.f;
    csync();
}

__device__ __noinline__ void poly_activation(const Ctx& c, const MkbhLayer& L) {
    const MkbhGlobals& g = *c.g;
    const int tid = threadIdx.x, K = L.ff;
    float s[3] = {0.f, 0.f, 0.f};
#pragma unroll 4
    for (int i = tid; i < K; i += kConsumers) {
        const float z = ld_cg_f32(g.proj + i), a = z * z;
        c.act[i] = z;
        s[0] += a;
        s[1] += a * a;
        s[2] += a * a * a;
    }
    csum<3>(c, s);
    const float f1 = L.act[0] / sqrtf(s[0] / K + g.eps), f2 = L.act[1] / sqrtf(s[1] / K + g.eps),
                f3 = L.act[2] / sqrtf(s[2] / K + g.eps), e = L.act[3];
    for (int i = tid; i < K; i += kConsumers) {
        const float z = c.act[i];
        c.act[i] = z * (f1 + z * (f2 + z * f3)) + e;
    }
    for (int i = K + tid; i < pad8(K); i += kConsumers) c.act[i] = 0.f;
    csync();
}

// ---- generalized delta rule: one step for a block of value columns of one head --------------- //
__device__ __noinline__ bool delta_step(Ctx& c, const int* w) {
    const MkbhGlobals& g = *c.g;
    const int layer = __ldg(w + 1), head = __ldg(w + 2), col0 = __ldg(w + 3), cols = __ldg(w + 4) - col0;
    const MkbhLayer& L = g.layers_device[layer];
    const int D = L.dim, HD = L.heads * D, R = L.rank, tid = threadIdx.x;
    const int parts = min(kMaxStateRows, kConsumers / cols);
    const int col = tid % cols, part = tid / cols;
    const bool live = part < parts;
    float* state = L.state + ((size_t)g.slot * L.heads + head) * D * D + col0 + col;
    float S[kMaxStateRows];
#pragma unroll
    for (int j = 0; j < kMaxStateRows; ++j) {
        const int i = part + j * parts;
        S[j] = (live && i < D && c.pos > 0) ? state[(size_t)i * D] : 0.f;
    }
    // scratch: w2 [D][R + 1], inner [R], r k a w rw ck [D] each, partial sums [2][parts][cols]
    float* w2 = c.act;
    float* inner = w2 + D * (R + 1);
    float *vr = inner + R, *vk = vr + D, *va = vk + D, *vw = va + D, *vrw = vw + D, *vck = vrw + D, *ps = vck + D;
    for (int i = tid; i < D * R; i += kConsumers)
        w2[(i / R) * (R + 1) + i % R] = __ldg(L.decay_w2 + (size_t)head * D * R + i);

    if (!wait_phase(c, layer, MKBH_OP_NORM_PROJ)) return false;
    rec(c, 1);
    for (int i = tid; i < R; i += kConsumers) inner[i] = tanhf(ld_cg_f32(g.proj + 5 * HD + i));
    for (int i = tid; i < 3 * D; i += kConsumers) {
        const int which = i / D, j = i % D;
        const float x = ld_cg_f32(g.proj + (which == 2 ? 3 : which) * HD + head * D + j);
        if (which == 2) va[j] = sigmoid_f(x);
        else (which ? vk : vr)[j] = x;
    }
    const float v = live ? ld_cg_f32(g.proj + 2 * HD + head * D + col0 + col) : 0.f;
    csync();
    // decays: four threads per channel
    for (int i = tid >> 2; i < D; i += kConsumers / 4) {  // uniform over the four threads
        float s = 0.f;
        for (int r = tid & 3; r < R; r += 4) s = fmaf(w2[i * (R + 1) + r], inner[r], s);
        const unsigned m = 0xfu << (tid & 28);
        s += __shfl_xor_sync(m, s, 1);
        s += __shfl_xor_sync(m, s, 2);
        if ((tid & 3) == 0) {
            const float d = expf(-L.decay_scale * sigmoid_f(s + __ldg(L.decay_w0 + head * D + i)));
            vw[i] = d;
            vrw[i] = vr[i] * d;
        }
    }
    // every warp: |k|^2, r . (a k), r . k
    float kk = 0.f, rak = 0.f, rk = 0.f;
    for (int i = tid & 31; i < D; i += 32) {
        const float k = vk[i], x = vr[i] * k;
        kk = fmaf(k, k, kk);
        rk += x;
        rak = fmaf(x, va[i], rak);
    }
    kk = warp_sum(kk);
    rk = warp_sum(rk);
    rak = warp_sum(rak);
    const float inv = 1.f / (kk + L.unit_eps);
    for (int i = tid; i < D; i += kConsumers) vck[i] = va[i] * vk[i] * inv;
    csync();
    float q = 0.f, o = 0.f;
#pragma unroll
    for (int j = 0; j < kMaxStateRows; ++j) {
        const int i = part + j * parts;
        if (live && i < D) {
            q = fmaf(vk[i], S[j], q);
            o = fmaf(vrw[i], S[j], o);
        }
    }
    if (live) {
        ps[part * cols + col] = q;
        ps[(parts + part) * cols + col] = o;
    }
    csync();
    if (live) {
        q = o = 0.f;
        for (int k = 0; k < parts; ++k) {
            q += ps[k * cols + col];
            o += ps[(parts + k) * cols + col];
        }
        if (part == 0) g.mixed[head * D + col0 + col] = o - rak * inv * q + rk * v;
#pragma unroll
        for (int j = 0; j < kMaxStateRows; ++j) {
            const int i = part + j * parts;
            if (i < D) state[(size_t)i * D] = fmaf(vk[i], v, fmaf(-vck[i], q, vw[i] * S[j]));
        }
    }
    signal_phase(c, layer, MKBH_OP_DELTA_STEP);
    return true;
}
__host__ __device__ inline int delta_scratch_floats(int dim, int rank) {
    return dim * (rank + 1) + rank + 6 * dim + 2 * kConsumers;
}

// ---- windowed differential attention: one split of the keys of one KV head -------------------- //
struct AttnScratch {  // float offsets; the key and value tiles follow
    int q, p, m, l, f, tile;
    __host__ __device__ AttnScratch(int nq, int dim, int chunk) {
        q = 0;
        p = nq * dim;
        p = (p + 3) & ~3;
        m = p + nq * chunk;
        l = m + nq;
        f = l + nq;
        tile = (f + nq + 3) & ~3;
    }
};
template <typename T>
__host__ __device__ inline int key_stride(int dim) {  // bytes; an odd number of 16-byte units
    const int u = (2 * dim * (int)sizeof(T) + 15) / 16;
    return (u | 1) * 16;
}
template <typename T>
__host__ __device__ inline int attn_scratch_bytes(int nq, int dim, int vdim, int chunk) {
    return AttnScratch(nq, dim, chunk).tile * 4 + chunk * (key_stride<T>(dim) + vdim * (int)sizeof(T)) + 16;
}

template <typename T>
__device__ __noinline__ bool attention_split(Ctx& c, const int* w) {
    const MkbhGlobals& g = *c.g;
    const int layer = __ldg(w + 1), kvh = __ldg(w + 2), split = __ldg(w + 3), splits = __ldg(w + 4);
    const MkbhLayer& L = g.layers_device[layer];
    const int D = L.dim, E = L.vdim, G = L.kv_heads, per = L.heads / G, nq = 2 * per;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, KC = c.p->attn_chunk;
    const AttnScratch a(nq, D, KC);
    float *q = c.act + a.q, *p = c.act + a.p, *m = c.act + a.m, *l = c.act + a.l, *f = c.act + a.f;
    T* kt = reinterpret_cast<T*>(c.act + a.tile);
    const int ks = key_stride<T>(D) / (int)sizeof(T);
    T* vt = kt + (size_t)KC * ks;

    const KeyRange keys(c.pos, L.window, L.keep_first);
    const int t_lo = (int)((long long)keys.count * split / splits), t_hi = (int)((long long)keys.count * (split + 1) / splits);
    const size_t rows0 = (size_t)g.slot * (L.cache_keep + L.cache_ring);
    T* kc = static_cast<T*>(L.k_cache) + rows0 * G * 2 * D + (size_t)kvh * 2 * D;
    T* vc = static_cast<T*>(L.v_cache) + rows0 * G * E + (size_t)kvh * E;
    // Rows of older positions: they do not depend on this step (other layers' caches included).
    auto stage_rows = [&](int c0, int nk) {
        const bool wide = (2 * D * sizeof(T)) % 16 == 0 && (E * sizeof(T)) % 16 == 0;
        const int unit = wide ? 16 / (int)sizeof(T) : 1;
        const int kn = 2 * D / unit, vn = E / unit;
        for (int i = tid; i < nk * (kn + vn); i += kConsumers) {
            const int t = i / (kn + vn), o = i % (kn + vn), j = keys.key(t_lo + c0 + t);
            if (j == c.pos) continue;
            const size_t row = cache_row(j, L.cache_keep, L.cache_ring);
            const T* src = o < kn ? kc + row * G * 2 * D + o * unit : vc + row * G * E + (o - kn) * unit;
            T* dst = o < kn ? kt + t * ks + o * unit : vt + t * E + (o - kn) * unit;
            if (wide) *reinterpret_cast<uint4*>(dst) = mkb::ld_cg_v4(src);
            else *dst = __ldcg(src);
        }
    };
    const int n0 = min(KC, t_hi - t_lo);
    stage_rows(0, n0);
    for (int i = tid; i < nq; i += kConsumers) {
        m[i] = -INFINITY;
        l[i] = 0.f;
    }
    if (!wait_phase(c, layer, MKBH_OP_NORM_PROJ)) return false;
    rec(c, 1);
    for (int i = tid; i < nq * D; i += kConsumers) q[i] = ld_cg_f32(g.proj + (size_t)kvh * nq * D + i);
    const int lanes_e = kConsumers / E;  // query vectors served side by side (E <= 512)
    const int e = tid % E, qv0 = tid / E;
    const bool has_e = qv0 < lanes_e;
    float acc[kMaxAcc];
#pragma unroll
    for (int i = 0; i < kMaxAcc; ++i) acc[i] = 0.f;

    for (int c0 = 0; c0 < t_hi - t_lo; c0 += KC) {
        const int nk = min(KC, t_hi - t_lo - c0);
        if (c0 > 0) stage_rows(c0, nk);
        if (keys.key(t_lo + c0 + nk - 1) == c.pos) {  // this token's own row (always the last key)
            const int t = nk - 1;
            const size_t row = cache_row(c.pos, L.cache_keep, L.cache_ring);
            for (int i = tid; i < 2 * D + E; i += kConsumers) {
                const bool is_k = i < 2 * D;
                T* cell = is_k ? kc + row * G * 2 * D + i : vc + row * G * E + (i - 2 * D);
                T x;
                if (L.owns_kv) {
                    const int off = L.heads * (2 * D + E) + (is_k ? kvh * 2 * D + i : G * 2 * D + kvh * E + (i - 2 * D));
                    x = from_f<T>(ld_cg_f32(g.proj + off));
                    *cell = x;
                } else {
                    x = __ldcg(cell);
                }
                if (is_k) kt[t * ks + i] = x;
                else vt[t * E + (i - 2 * D)] = x;
            }
        }
        csync();
        // scores: consecutive threads take consecutive keys of one query vector
        for (int i = tid; i < nq * KC; i += kConsumers) {
            const int t = i % KC, qv = i / KC;
            float s = -INFINITY;
            if (t < nk) {
                const T* k = kt + t * ks + (qv & 1) * D;
                const float* qq = q + qv * D;
                s = 0.f;
                int d = 0;
                if ((D * sizeof(T)) % 16 == 0) {
                    constexpr int U = Chunk<T>::kElems;
                    for (; d < D; d += U) s = Chunk<T>::dot(lds_v4(smem_u32(k + d)), qq + d, s);
                } else {
                    for (; d < D; ++d) s = fmaf(to_f(k[d]), qq[d], s);
                }
                s *= L.scale;
            }
            p[qv * KC + t] = s;
        }
        csync();
        for (int qv = warp; qv < nq; qv += kConsumerWarps) {
            float x = -INFINITY;
            for (int t = lane; t < KC; t += 32) x = fmaxf(x, p[qv * KC + t]);
            x = fmaxf(warp_max(x), m[qv]);
            float s = 0.f;
            for (int t = lane; t < KC; t += 32) {
                const float y = expf(p[qv * KC + t] - x);
                p[qv * KC + t] = y;
                s += y;
            }
            s = warp_sum(s);
            if (lane == 0) {
                const float fac = expf(m[qv] - x);
                f[qv] = fac;
                l[qv] = l[qv] * fac + s;
                m[qv] = x;
            }
            __syncwarp();
        }
        csync();
        if (has_e) {
#pragma unroll
            for (int i = 0; i < kMaxAcc; ++i) {
                const int qv = qv0 + i * lanes_e;
                if (qv < nq) acc[i] *= f[qv];
            }
            for (int t = 0; t < nk; t += 4) {  // weights beyond nk are zero
                float v[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) v[j] = t + j < nk ? to_f(vt[(t + j) * E + e]) : 0.f;
#pragma unroll
                for (int i = 0; i < kMaxAcc; ++i) {
                    const int qv = qv0 + i * lanes_e;
                    if (qv < nq) {
                        const float4 w4 = *reinterpret_cast<const float4*>(p + qv * KC + t);
                        acc[i] = fmaf(w4.x, v[0], fmaf(w4.y, v[1], fmaf(w4.z, v[2], fmaf(w4.w, v[3], acc[i]))));
                    }
                }
            }
        }
        csync();
    }
    // partial rows [head][map][split][m, l, acc...]
    const int PE = g.part_vdim + 2;
    float* part = g.attn_part + (size_t)kvh * nq * g.max_splits * PE;
    if (has_e) {
#pragma unroll
        for (int i = 0; i < kMaxAcc; ++i) {
            const int qv = qv0 + i * lanes_e;
            if (qv < nq) {
                float* row = part + ((size_t)qv * g.max_splits + split) * PE;
                row[2 + e] = acc[i];
                if (e == 0) {
                    row[0] = m[qv];
                    row[1] = l[qv];
                }
            }
        }
    }
    csync();
    if (tid == 0) {
        int old;
        int* cnt = g.counters + 2 + (g.num_layers + 1) * MKBH_BARRIERS_PER_LAYER + layer * g.max_kv_heads + kvh;
        asm volatile("atom.acq_rel.gpu.global.add.s32 %0, [%1], 1;" : "=r"(old) : "l"(cnt) : "memory");
        c.ctl[1] = old == splits - 1;
    }
    csync();
    if (!c.ctl[1]) return true;
    // the split of this KV head that arrives last merges the partial rows
    for (int hh = warp; hh < per; hh += kConsumerWarps) {
        float fac[2], inv[2];
        const float* src[2];
        for (int b = 0; b < 2; ++b) {
            src[b] = part + (size_t)(2 * hh + b) * g.max_splits * PE;
            float ms = lane < splits ? ld_cg_f32(src[b] + (size_t)lane * PE) : -INFINITY;
            const float ls = lane < splits ? ld_cg_f32(src[b] + (size_t)lane * PE + 1) : 0.f;
            const float M = warp_max(ms);
            fac[b] = expf(ms - M);
            inv[b] = 1.f / warp_sum(ls * fac[b]);
        }
        const int h = kvh * per + hh;
        float* o = c.act + (size_t)warp * E;  // q, p and the tiles are no longer needed
        float sq = 0.f;
        for (int e2 = lane; e2 - lane < E; e2 += 32) {  // uniform trip count: the loop shuffles
            float a1 = 0.f, a2 = 0.f;
            for (int s = 0; s < splits; ++s) {
                const float f1 = __shfl_sync(0xffffffffu, fac[0], s), f2 = __shfl_sync(0xffffffffu, fac[1], s);
                if (e2 < E) {
                    a1 = fmaf(f1, ld_cg_f32(src[0] + (size_t)s * PE + 2 + e2), a1);
                    a2 = fmaf(f2, ld_cg_f32(src[1] + (size_t)s * PE + 2 + e2), a2);
                }
            }
            if (e2 < E) {
                const float x = a1 * inv[0] - L.lambda * (a2 * inv[1]);
                o[e2] = x;
                sq += x * x;
            }
        }
        const float fin = (1.f - L.diff) / sqrtf(warp_sum(sq) / E + g.eps);
        for (int e2 = lane; e2 < E; e2 += 32)
            g.mixed[h * E + e2] = o[e2] * fin * sigmoid_f(ld_cg_f32(g.proj + L.heads * 2 * D + h * E + e2));
    }
    signal_phase(c, layer, MKBH_OP_ATTENTION);
    return true;
}

// ---- output head: running argmax --------------------------------------------------------------- //
__device__ __forceinline__ unsigned long long argmax_key(float v, int i) {
    uint32_t u = __float_as_uint(v);
    u = (u >> 31) ? ~u : (u | 0x80000000u);
    return ((unsigned long long)u << 32) | (0xffffffffu - (uint32_t)i);
}

template <typename T>
__device__ bool run_instruction(Ctx& c, const int* w) {
    const MkbhGlobals& g = *c.g;
    const int op = __ldg(w), layer = __ldg(w + 1), tid = threadIdx.x;
    if (op == MKBH_OP_DELTA_STEP) return delta_step(c, w);
    if (op == MKBH_OP_ATTENTION) return attention_split<T>(c, w);
    Block b;
    if (!weight_block<T>(g, w, b)) {
        if (tid == 0) report(c, MKBH_ERR_BAD_OPCODE, 1, op, 0, 0);
        csync();
        return false;
    }
    const MkbhLayer& L = g.layers_device[op == MKBH_OP_HEAD ? 0 : layer];
    int groups = 1;
    switch (op) {
        case MKBH_OP_NORM_PROJ: {
            if (layer > 0 && !wait_phase(c, layer - 1, last_phase(g.layers_device[layer - 1]))) return false;
            rec(c, 1);
            norm_activation<T>(c, L.norm1, layer == 0, layer == 0 && b.r0 == 0);
            rec(c, 2);
            if (!matvec<T>(c, b, groups)) return false;
            for (int i = tid; i < b.r1 - b.r0; i += kConsumers)
                g.proj[b.r0 + i] = row_sum(c, i, groups) + (L.in_bias ? __ldg(L.in_bias + b.r0 + i) : 0.f);
        } break;
        case MKBH_OP_OUT_PROJ:
        case MKBH_OP_DOWN: {
            const bool down = op == MKBH_OP_DOWN;
            const float* ls = down ? L.ls2 : L.ls1;
            const int prev = down ? MKBH_OP_NORM_UP : L.mixer == MKBH_DELTA_RULE ? MKBH_OP_DELTA_STEP : MKBH_OP_ATTENTION;
            if (!wait_phase(c, layer, prev)) return false;
            rec(c, 1);
            if (down) poly_activation(c, L);
            else mixed_activation(c, L);
            rec(c, 2);
            if (!matvec<T>(c, b, groups)) return false;
            for (int i = tid; i < b.r1 - b.r0; i += kConsumers) {
                float* x = g.x + b.r0 + i;  // this instruction is the only writer of its rows
                *x = fmaf(__ldg(ls + b.r0 + i), row_sum(c, i, groups), ld_cg_f32(x));
            }
        } break;
        case MKBH_OP_NORM_UP: {
            if (!wait_phase(c, layer, MKBH_OP_OUT_PROJ)) return false;
            rec(c, 1);
            norm_activation<T>(c, L.norm2, false, false);
            rec(c, 2);
            if (!matvec<T>(c, b, groups)) return false;
            // (the stacked projection is no longer needed: its buffer takes the feed-forward's input)
            for (int i = tid; i < b.r1 - b.r0; i += kConsumers) g.proj[b.r0 + i] = row_sum(c, i, groups);
        } break;
        default: {  // MKBH_OP_HEAD
            const int last = g.num_layers - 1;
            if (!wait_phase(c, last, last_phase(g.layers_device[last]))) return false;
            rec(c, 1);
            norm_activation<T>(c, g.final_norm, false, false);
            rec(c, 2);
            if (!matvec<T>(c, b, groups)) return false;
            unsigned long long best = 0;
            for (int i = tid; i < b.r1 - b.r0; i += kConsumers) {
                const float y = row_sum(c, i, groups);
                g.logits[b.r0 + i] = y;
                const unsigned long long k = argmax_key(y, b.r0 + i);
                best = k > best ? k : best;
            }
            if (g.argmax_out != nullptr) {
#pragma unroll
                for (int o = 16; o; o >>= 1) {
                    const unsigned long long k = __shfl_xor_sync(0xffffffffu, best, o);
                    best = k > best ? k : best;
                }
                unsigned long long* total = reinterpret_cast<unsigned long long*>(g.counters);
                if ((tid & 31) == 0 && best) atomicMax(total, best);
                csync();
                if (tid == 0) {
                    int old;
                    asm volatile("atom.acq_rel.gpu.global.add.s32 %0, [%1], 1;"
                                 : "=r"(old)
                                 : "l"(counter(c, g.num_layers, MKBH_OP_HEAD))
                                 : "memory");
                    if (old == threshold(c, g.num_layers, MKBH_OP_HEAD) - 1)
                        *g.argmax_out = (int)(0xffffffffu - (uint32_t)(atomicMax(total, 0ull) & 0xffffffffull));
                }
                return true;
            }
        } break;
    }
    signal_phase(c, op == MKBH_OP_HEAD ? g.num_layers : layer, op);
    return true;
}

template <typename T>
__global__ void __launch_bounds__(kBlock, 1) hybrid_decode_kernel(const __grid_constant__ Params p) {
    extern __shared__ uint8_t raw[];
    const uint32_t raw32 = smem_u32(raw), base = (raw32 + 127u) & ~127u;
    uint8_t* gb = raw + (base - raw32);
    const Smem sm(p.stages, p.act_bytes);
    Ctx c;
    c.p = &p;
    c.g = &p.g;
    c.base = base;
    c.act = reinterpret_cast<float*>(gb + sm.act);
    c.part = reinterpret_cast<float*>(gb + sm.part);
    c.red = reinterpret_cast<float*>(gb + sm.red);
    c.bars = base + sm.bars;
    c.ctl = reinterpret_cast<volatile int*>(gb + sm.ctl);
    c.instr = -1;
    c.opcode = -1;
    c.slot = 0;
    c.phase = 0;
    c.pos = p.g.pos_device ? __ldg(p.g.pos_device) : p.g.pos0;
    if (threadIdx.x == 0) {
        for (int s = 0; s < p.stages; ++s) {
            mbar_init(c.full(s), 1);
            mbar_init(c.empty(s), kConsumerWarps);
        }
        c.ctl[0] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    __syncthreads();
    if (c.pos < 0 || c.pos >= p.g.max_positions) {  // uniform over the grid
        if (threadIdx.x == 0) report(c, MKBH_ERR_INVALID_ARGUMENT, 1, c.pos, p.g.max_positions, 0);
        return;
    }
    if (threadIdx.x < kConsumers) {
        const int* queue = p.g.instructions + (size_t)blockIdx.x * p.g.queue_len * MKBH_INTS_PER_INSTRUCTION;
        for (int i = 0; i < p.g.queue_len; ++i) {
            const int* w = queue + (size_t)i * MKBH_INTS_PER_INSTRUCTION;
            c.instr = i;
            c.opcode = __ldg(w);
            if (c.opcode == MKBH_OP_NOOP) continue;
            rec(c, 0);
            if (!run_instruction<T>(c, w)) break;
            rec(c, 4);
        }
    } else if (threadIdx.x == kConsumers) {
        loader_main<T>(c);
    }
    __syncthreads();
}

template <typename T>
cudaError_t launch(const MkbhGlobals& g, cudaStream_t s) {
    Params p;
    p.g = g;
    p.timeout_ns = (g.wait_timeout_ms ? g.wait_timeout_ms : 2000u) * 1000000ull;
    if (!(g.flags & MKBH_FLAG_RECORD_TIMINGS)) p.g.timings = nullptr;
    int act = 4 * pad8(g.width);
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        const bool delta = L.mixer == MKBH_DELTA_RULE;
        int need = 4 * pad8(L.heads * (delta ? L.dim : L.vdim));
        if (delta) need = max(need, 4 * delta_scratch_floats(L.dim, L.rank));
        if (L.ff) need = max(need, 4 * pad8(L.ff));
        act = max(act, need);
    }
    act = max(act, kScratchMin);
    // keys staged at a time: 64, fewer when a tile of wide heads would not fit
    p.attn_chunk = 64;
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        if (L.mixer != MKBH_DIFF_ATTENTION) continue;
        const int nq = 2 * (L.heads / L.kv_heads);
        act = max(act, 4 * kConsumerWarps * L.vdim);  // merged rows
        act = max(act, attn_scratch_bytes<T>(nq, L.dim, L.vdim, 8));
        while (p.attn_chunk > 8 && attn_scratch_bytes<T>(nq, L.dim, L.vdim, p.attn_chunk) > act) p.attn_chunk -= 8;
    }
    p.act_bytes = (act + 127) & ~127;
    const int fixed = Smem(0, p.act_bytes).total + 128;
    p.stages = (kSmemLimit - fixed) / kStage;
    if (p.stages > kMaxStages) p.stages = kMaxStages;
    if (p.stages < 2) return cudaErrorInvalidValue;
    p.l2_window = p.stages + 8;
    const int smem = Smem(p.stages, p.act_bytes).total + 128;
    static int set[64] = {};
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    if (set[dev & 63] < smem) {
        e = cudaFuncSetAttribute(hybrid_decode_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return e;
        set[dev & 63] = smem;
    }
    e = cudaMemsetAsync(g.counters, 0, (size_t)g.num_counters * 4, s);
    if (e != cudaSuccess) return e;
    // cooperative: the CTAs wait for one another, so all of them must be resident
    void* args[] = {&p};
    return cudaLaunchCooperativeKernel((const void*)hybrid_decode_kernel<T>, dim3(g.num_sms), dim3(kBlock), args,
                                       (size_t)smem, s);
}

}  // namespace

cudaError_t decode_launch(const MkbhGlobals& g, cudaStream_t s) {
    return g.dtype == MKBH_F32 ? launch<float>(g, s) : launch<bf16>(g, s);
}

}  // namespace mkbh
