// Decode megakernel of the hybrid models: one token of one sequence in one persistent launch.
//
// The scheme of megakernel.cu - one CTA per SM, an instruction queue per CTA, a ring of weight
// stages in shared memory that a loader thread keeps full across instruction boundaries, counters
// in HBM that order the phases - for layers that are listed one by one (delta-rule recurrence,
// windowed differential, rotary or latent attention, optional feed-forward) and for any sizes:
//   * a weight block is a run of whole rows, contiguous in memory, so a stage is ONE untiled bulk
//     copy (no tensor maps, no divisibility rules beyond the zero padding of a row to 16 bytes);
//   * 16 consumer warps multiply from shared memory with fp32 FMA (batch 1 is bandwidth-bound), the
//     same code for bf16 and float weights; every warp owns a fixed slice of the input columns, whose
//     activations stay in registers for the whole instruction;
//   * every output row has exactly one owner, which also adds it to the 32-bit residual stream: no
//     atomics on data, bit-identical results from run to run;
//   * an operand warp runs one instruction ahead: it fetches the next instruction's words, its layer
//     descriptor and its vectors (norm weights, layer scales, biases, decay factors) into shared
//     memory, so that no pointer or vector is chased through HBM on the critical path;
//   * what else does not depend on the token (recurrent state, older keys and values) is fetched
//     before an instruction waits for its producers;
//   * every wait is bounded and reports into the status record.
//
// Compiled once per set of mechanisms (MKBH_FEATURES, see Features): hybrid_decode_rotary.cu and
// hybrid_decode_mixed.cu include this file.
#include "hybrid_kernels.h"

#ifndef MKBH_FEATURES
#define MKBH_FEATURES 1
#endif

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
constexpr int kOperandWarp = kConsumerWarps + 1;  // (warp 16 is the loader)
// The release of a counter waits until the CTA's stores are visible to the GPU.  Where an instruction's
// successor in the queue is often independent of it (feed-forwards beside mixers), a warp of its own
// does that, so that the consumers go on.
constexpr bool kSignalWarp = (MKBH_FEATURES & 2) != 0;
constexpr int kSignals = 4;  // signals in flight
constexpr int kBlock = kConsumers + (kSignalWarp ? 96 : 64);
constexpr int kStage = 32768;
static_assert(kStage >= kMaxRowBytes, "a stage holds whole rows");
constexpr int kMaxStages = 6;
constexpr int kPartFloats = 4096;      // per-row, per-column-group partial sums of an instruction
constexpr int kMaxRows = 512;          // output rows of an instruction
static_assert(kPartFloats * 4 <= 40 * 1024, "");
constexpr int kScratchMin = 40 * 1024; // activation / mixer scratch, at least
constexpr int kRowVecBytes = kMaxRows * 4 + 32;
constexpr int kSmemLimit = 226 * 1024;
constexpr int kMaxStash = 512;         // channels whose normalised input an instruction publishes
constexpr int kMaxChannels = 8;        // key channels of one column a lane carries (dim <= 256)

// Which mechanisms a build of the kernel has; a launch takes the smallest build that serves its
// layers, so that one family's code and registers do not weigh on the other's.
enum Features {
    kClassic = 1,  // delta rule, differential attention, PolyNorm, layer norms
    kRotary = 2,   // rotary and latent attention, gated units, feed-forwards beside mixers, convolutions, loops
};

struct Params {
    MkbhGlobals g;
    int stages, act_bytes, vec_bytes;
    int attn_chunk;        // keys staged at a time
    int last_buf;          // residual buffer of the last layer
    int part_base;         // where the second vector of an instruction lies in the vector buffer
    unsigned long long timeout_ns;
};

// What the operand warp prepares for one instruction.
struct Desc {
    int op, layer, a0, a1, a2;
    int wait_idx, wait_thr;   // phase counter to wait for (index -1: none)
    int arrive_idx, arrive_thr;
    int row_bytes, per_stage, groups;
    int has_vec, vec_off, row_off;  // vector operands: present, byte offsets inside their buffers
    int part_off;                   // second vector (terms of earlier inputs), -1: none
    MkbhLayer L;
};
static_assert(sizeof(MkbhLayer) % 8 == 0, "");
constexpr int kDescBytes = (sizeof(Desc) + 127) & ~127;

enum Bar { kDescFull = 0, kDescEmpty = 2, kVecFull = 4, kVecEmpty = 5, kSigFull = 6, kSigEmpty = kSigFull + kSignals, kRing = kSigEmpty + kSignals };

struct Smem {  // byte offsets from the 128-byte aligned base
    int act, vec, rows, desc, red, stash, layer, bars, ctl, total;
    __host__ __device__ Smem(int stages, int act_bytes, int vec_bytes) {
        act = stages * kStage;          // activations; partial sums once they are in registers
        vec = act + act_bytes;          // norm weights / decay factor
        rows = vec + vec_bytes;         // two slots: per-row vectors (bias, layer scale, decay bias)
        desc = rows + 2 * kRowVecBytes;
        red = (desc + 2 * kDescBytes + 127) & ~127;
        stash = red + 2 * 3 * kConsumerWarps * 4;
        layer = stash + kMaxStash * 4;  // the loader's copy of a layer descriptor
        bars = layer + (int)((sizeof(MkbhLayer) + 15) & ~15);
        ctl = bars + (kRing + 2 * kMaxStages) * 8;
        total = ctl + 16 * 4;  // (words 8.. are the signals' counters)
    }
};

struct Cta {  // small and passed by reference to inlined code only: stays in registers
    uint32_t base, bars;
    uint8_t* gb;
    volatile int* ctl;  // [0] CTA abort, [1] last-arriver verdict, [2], [3] agreed abort
    int instr, opcode, pos, turn, signals;
    __device__ __forceinline__ uint32_t bar(int i) const { return bars + i * 8; }
    __device__ __forceinline__ uint32_t full(int s) const { return bars + (kRing + s) * 8; }
    __device__ __forceinline__ uint32_t empty(int s) const { return bars + (kRing + kMaxStages + s) * 8; }
};

__device__ __forceinline__ void csync() { asm volatile("bar.sync 1, %0;" ::"n"(kConsumers) : "memory"); }

__device__ __noinline__ void report(int* st, volatile int* ctl, int code, int role, int instr, int op, int d0, int d1, int d2) {
    if (atomicCAS(&st[0], 0, code) == 0) {
        st[1] = blockIdx.x;
        st[2] = instr;
        st[3] = op;
        st[4] = role;
        st[5] = d0;
        st[6] = d1;
        st[7] = d2;
        __threadfence();
    }
    atomicExch(&st[15], 1);
    ctl[0] = 1;
}

__device__ __noinline__ bool bar_wait_slow(uint32_t bar, uint32_t parity, volatile int* ctl, int* status,
                                           unsigned long long timeout_ns, int role, int instr, int op, bool honour_abort) {
    const unsigned long long t0 = globaltimer_ns();
    for (uint32_t spins = 1;; ++spins) {
        if (mbar_try_wait(bar, parity)) return true;
        if ((spins & 63u) == 0) {
            if (honour_abort && ctl[0]) return false;
            if (globaltimer_ns() - t0 > timeout_ns) {
                report(status, ctl, MKBH_ERR_DEVICE_TIMEOUT, role, instr, op, -1, 0, 0);
                return false;
            }
        }
    }
}
__device__ __forceinline__ bool bar_wait(const Params& p, const Cta& c, uint32_t bar, uint32_t parity, int role,
                                         bool honour_abort = true) {
    return mbar_try_wait(bar, parity) ||
           bar_wait_slow(bar, parity, c.ctl, p.g.status, p.timeout_ns, role, c.instr, c.opcode, honour_abort);
}

// One consumer thread's view of the abort word for all of them (the loaders may set it at any
// time): true if they go on together.
__device__ __forceinline__ bool agree(Cta& c) {
    // two words in turn: a slow thread may still read the previous verdict while the next is written
    const int w = 2 + (c.turn++ & 1);
    if (threadIdx.x == 0) c.ctl[w] = c.ctl[0];
    csync();
    return c.ctl[w] == 0;
}

__device__ __noinline__ void poll_counter(const int* addr, int thr, volatile int* ctl, int* status,
                                          unsigned long long timeout_ns, int instr, int op) {
    unsigned long long t0 = 0;
    uint32_t spins = 0;
    while (ld_acquire_gpu(addr) < thr) {
        if ((++spins & 63u) == 0) {
            if (ctl[0]) return;
            if (*reinterpret_cast<volatile int*>(&status[15])) {
                ctl[0] = 1;
                return;
            }
            const unsigned long long now = globaltimer_ns();
            if (t0 == 0) t0 = now;
            else if (now - t0 > timeout_ns) {
                report(status, ctl, MKBH_ERR_DEVICE_TIMEOUT, 1, instr, op, thr, ld_acquire_gpu(addr), 0);
                return;
            }
        }
        __nanosleep(20);
    }
}

// Consumer thread 0, behind a consumer barrier: count an instruction's end into a phase counter
// (-1: no more of them).
__device__ __forceinline__ void post_signal(const Params& p, Cta& c, int* counters, int idx) {
    if constexpr (kSignalWarp) {
        const int slot = c.signals % kSignals;
        bar_wait(p, c, c.bar(kSigEmpty + slot), ((c.signals / kSignals) & 1u) ^ 1u, 1);
        c.ctl[8 + slot] = idx;
        mbar_arrive(c.bar(kSigFull + slot));
        ++c.signals;
    } else if (idx >= 0) {
        red_release_gpu_add(counters + idx, 1);
    }
}
__device__ __forceinline__ void signal_main(const Params& p, Cta& c) {
    int* counters = p.g.counters + 2;
    for (;; ++c.signals) {
        const int slot = c.signals % kSignals;
        if (!bar_wait(p, c, c.bar(kSigFull + slot), (c.signals / kSignals) & 1u, 3)) return;
        const int idx = c.ctl[8 + slot];
        if (idx < 0) return;
        red_release_gpu_add(counters + idx, 1);
        mbar_arrive(c.bar(kSigEmpty + slot));
    }
}

__device__ __forceinline__ int phase_index(int layer, int op) { return layer * MKBH_BARRIERS_PER_LAYER + op; }

// Float buffers beside the stacked projection: feed-forward input and output of parallel layers,
// absorbed queries.
__device__ __forceinline__ float* side_in(const MkbhGlobals& g) { return g.side; }
__device__ __forceinline__ float* side_out(const MkbhGlobals& g) { return g.side + g.side_ff; }
__device__ __forceinline__ float* side_query(const MkbhGlobals& g) { return side_out(g) + pad8(g.width); }

// ---- the weight stream --------------------------------------------------------------------- //
struct Block {  // rows [r0, r1) of a matrix of `row_bytes` rows
    const uint8_t* w;
    int r0, r1, row_bytes;
};
template <typename T>
__device__ __forceinline__ bool weight_block(const MkbhGlobals& g, int op, const MkbhLayer* L, int r0, int r1, Block& b) {
    int K;
    switch (op) {
        case MKBH_OP_NORM_PROJ: b.w = (const uint8_t*)L->in_w; K = g.width; break;
        case MKBH_OP_OUT_PROJ:
            b.w = (const uint8_t*)L->out_w;
            K = mixer_out(*L);
            break;
        case MKBH_OP_NORM_UP: b.w = (const uint8_t*)L->up_w; K = g.width; break;
        case MKBH_OP_DOWN: b.w = (const uint8_t*)L->down_w; K = L->ff; break;
        case MKBH_OP_HEAD: b.w = (const uint8_t*)g.head; K = g.width; break;
#if MKBH_FEATURES & 2
        case MKBH_OP_ENTER: b.w = (const uint8_t*)L->enter_w; K = 2 * g.width; break;
        case MKBH_OP_ABSORB: b.w = (const uint8_t*)L->absorb_w; K = L->dim; break;
        case MKBH_OP_EXPAND:  // (behind the keys' rows)
            K = L->rank;
            b.w = (const uint8_t*)L->expand_w + (size_t)L->heads * L->dim * pad8(K) * sizeof(T);
            break;
#endif
        default: return false;
    }
    b.r0 = r0;
    b.r1 = r1;
    b.row_bytes = pad8(K) * (int)sizeof(T);
    return true;
}

template <typename T>
struct Cursor {  // the queue's weight blocks as a flat sequence of stages
    int i = 0, row = 0, per = 1;
    bool open = false;
    Block b;
    __device__ bool next(const MkbhGlobals& g, const int* queue, const uint8_t*& src, uint32_t& bytes) {
        while (!open) {
            if (i >= g.queue_len) return false;
            const int* w = queue + (size_t)i * MKBH_INTS_PER_INSTRUCTION;
            const int op = __ldg(w), layer = __ldg(w + 1);
            if (weight_block<T>(g, op, g.layers_device + layer, __ldg(w + 2), __ldg(w + 3), b) && b.r1 > b.r0) {
                open = true;
                row = b.r0;
                per = kStage / b.row_bytes;
            } else {
                ++i;
            }
        }
        const int n = min(per, b.r1 - row);
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

// ---- operand warp ------------------------------------------------------------------------- //
// Column groups of an input of `chunks` 16-byte chunks: warps that share a row.
__host__ __device__ inline int column_groups(int chunks) {
    int n = 1;
    while (n < kConsumerWarps && n * 32 < chunks) n *= 2;
    return n;
}
// Phase that completes the residual stream a layer leaves.
__device__ __forceinline__ int last_phase(const MkbhLayer* L) {
    return __ldg(&L->ff) && !__ldg(&L->parallel) ? MKBH_OP_DOWN : MKBH_OP_OUT_PROJ;
}

__device__ __forceinline__ void copy_vec(uint32_t dst, const void* src, int bytes, uint32_t bar, uint64_t policy) {
    const uint64_t a = reinterpret_cast<uint64_t>(src) & ~15ull, e = (reinterpret_cast<uint64_t>(src) + bytes + 15) & ~15ull;
    mkb::tma_bulk_g2s(dst, reinterpret_cast<const void*>(a), (uint32_t)(e - a), bar, policy);
}
__device__ __forceinline__ uint32_t vec_span(const void* src, int bytes) {
    const uint64_t a = reinterpret_cast<uint64_t>(src);
    return (uint32_t)(((a + bytes + 15) & ~15ull) - (a & ~15ull));
}

template <typename T>
__device__ __forceinline__ void operand_main(const Params& p, Cta& c, const Smem& sm) {
    const MkbhGlobals& g = p.g;
    const int lane = threadIdx.x & 31;
    const int* queue = g.instructions + (size_t)blockIdx.x * g.queue_len * MKBH_INTS_PER_INSTRUCTION;
    const uint64_t policy = mkb::l2_policy_evict_first();
    uint32_t vecs = 0;  // vector operands issued
    int done = 0;       // descriptors published
    bool ok = true;
    for (int i = 0; i < g.queue_len && ok; ++i) {
        const int slot = i & 1;
        Desc* d = reinterpret_cast<Desc*>(c.gb + sm.desc + slot * kDescBytes);
        const int w = lane < 5 ? __ldg(queue + (size_t)i * MKBH_INTS_PER_INSTRUCTION + lane) : 0;
        const int op = __shfl_sync(0xffffffffu, w, 0), layer = __shfl_sync(0xffffffffu, w, 1);
        c.instr = i;
        c.opcode = op;
        int flag = 1;
        if (lane == 0) flag = bar_wait(p, c, c.bar(kDescEmpty + slot), ((i >> 1) & 1u) ^ 1u, 2);
        ok = __shfl_sync(0xffffffffu, flag, 0) != 0;
        if (!ok) break;
        if (lane < 5) (&d->op)[lane] = w;
        const uint2* src = reinterpret_cast<const uint2*>(g.layers_device + layer);
        for (int k = lane; k < (int)sizeof(MkbhLayer) / 8; k += 32) reinterpret_cast<uint2*>(&d->L)[k] = __ldg(src + k);
        __syncwarp();
        const void *vec = nullptr, *rows = nullptr, *part = nullptr;
        int vec_n = 0, row_n = 0, K = 0;
        if (lane == 0) {
            const MkbhLayer& L = d->L;
            const bool delta = L.mixer == MKBH_DELTA_RULE;
            int wl = layer, wop = 0;
            const bool latent = L.mixer == MKBH_LATENT_ATTENTION;
            // phase that completes the layer's input stream
            auto input_phase = [&](bool entered) {
                if (L.enter_w != nullptr && entered) {
                    wop = MKBH_OP_ENTER;
                } else {
                    wl = layer - 1;
                    wop = layer > 0 ? last_phase(g.layers_device + wl) : -1;
                }
            };
            switch (op) {
                case MKBH_OP_ENTER: K = 2 * g.width; input_phase(false); break;
                case MKBH_OP_NORM_PROJ:
                    K = g.width; vec_n = K * 4;
                    vec = L.canon_taps ? L.canon_gain : L.norm1;
                    if (L.canon_taps > 1 && c.pos > 0) part = L.canon_part + ((size_t)g.slot * 2 + (c.pos & 1)) * g.width;
                    rows = L.conv_taps ? L.conv_w + (size_t)(L.conv_taps - 1) * L.in_rows : L.in_bias;
                    input_phase(true);
                    break;
                case MKBH_OP_DELTA_STEP:
                    vec = (const uint8_t*)L.decay_w2 + (size_t)d->a0 * L.dim * L.rank * sizeof(T);
                    vec_n = L.dim * L.rank * (int)sizeof(T);
                    rows = L.decay_w0 + d->a0 * L.dim;
                    row_n = L.dim * 4;
                    wop = MKBH_OP_NORM_PROJ;
                    break;
                case MKBH_OP_ABSORB: K = L.dim; wop = MKBH_OP_NORM_PROJ; break;
                case MKBH_OP_ATTENTION: wop = latent ? MKBH_OP_ABSORB : MKBH_OP_NORM_PROJ; break;
                case MKBH_OP_EXPAND: K = L.rank; wop = MKBH_OP_ATTENTION; break;
                case MKBH_OP_OUT_PROJ:
                    K = mixer_out(L);
                    rows = L.ls1;
                    if (delta) vec = L.out_norm, vec_n = K * 4;
                    wop = mixer_phase(L.mixer);
                    break;
                case MKBH_OP_NORM_UP:
                    K = g.width; vec = L.norm2; vec_n = K * 4;
                    if (L.parallel) input_phase(true);
                    else wop = MKBH_OP_OUT_PROJ;
                    break;
                case MKBH_OP_DOWN: K = L.ff; rows = L.parallel ? nullptr : L.ls2; wop = MKBH_OP_NORM_UP; break;
                case MKBH_OP_HEAD:
                    K = g.width; vec = g.final_norm; vec_n = K * 4;
                    wl = g.num_layers - 1;
                    wop = last_phase(g.layers_device + wl);
                    break;
                default: wop = -1; break;
            }
            if (K > 0 && rows != nullptr) {
                rows = (const float*)rows + d->a0;
                row_n = (d->a1 - d->a0) * 4;
            }
            d->wait_idx = wop < 0 ? -1 : phase_index(wl, wop);
            d->wait_thr = wop < 0 ? 0 : __ldg(g.arrivals + phase_index(wl, wop));
            // (a feed-forward beside a mixer counts into the phase that the output projection waits for)
            d->arrive_idx = phase_index(op == MKBH_OP_HEAD ? g.num_layers : layer,
                                        op == MKBH_OP_DOWN && L.parallel ? mixer_phase(L.mixer) : op);
            d->arrive_thr = op == MKBH_OP_HEAD ? __ldg(g.arrivals + d->arrive_idx) : 0;
            d->row_bytes = pad8(K) * (int)sizeof(T);
            d->per_stage = K > 0 ? kStage / d->row_bytes : 0;
            d->groups = column_groups(d->row_bytes / 16);
            d->has_vec = vec != nullptr;
            d->vec_off = (int)(reinterpret_cast<uint64_t>(vec) & 15);
            d->part_off = part != nullptr ? p.part_base + (int)(reinterpret_cast<uint64_t>(part) & 15) : -1;
            d->row_off = rows != nullptr && row_n > 0 ? (int)(reinterpret_cast<uint64_t>(rows) & 15) : -1;
        }
        __syncwarp();
        if (lane == 0) {
            const uint32_t full = c.bar(kDescFull + slot);
            if (d->row_off >= 0) {
                mbar_expect_tx(full, vec_span(rows, row_n));
                copy_vec(c.base + sm.rows + slot * kRowVecBytes, rows, row_n, full, policy);
            } else {
                mbar_arrive(full);
            }
            if (vec != nullptr) {
                flag = bar_wait(p, c, c.bar(kVecEmpty), (vecs & 1u) ^ 1u, 2);
                if (flag) {
                    mbar_expect_tx(c.bar(kVecFull), vec_span(vec, vec_n) + (part != nullptr ? vec_span(part, vec_n) : 0u));
                    copy_vec(c.base + sm.vec, vec, vec_n, c.bar(kVecFull), policy);
                    if (part != nullptr) copy_vec(c.base + sm.vec + p.part_base, part, vec_n, c.bar(kVecFull), policy);
                    ++vecs;
                }
            }
        }
        done = i + 1;
        ok = __shfl_sync(0xffffffffu, flag, 0) != 0;
    }
    if (lane == 0) {  // nothing of it may be in flight at exit
        for (int i = done > 2 ? done - 2 : 0; i < done; ++i) bar_wait(p, c, c.bar(kDescFull + (i & 1)), (i >> 1) & 1u, 2, false);
        if (vecs > 0) bar_wait(p, c, c.bar(kVecFull), (vecs - 1) & 1u, 2, false);
    }
}

// ---- consumers ------------------------------------------------------------------------------ //
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
        float acc2 = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            acc = fmaf(mkb::bf16_lo(u[i]), a[2 * i], acc);
            acc2 = fmaf(mkb::bf16_hi(u[i]), a[2 * i + 1], acc2);
        }
        return acc + acc2;
    }
};

// Multiply the instruction's rows with the activations in `act` (fp32, zero beyond the matrix's
// columns); partial sums [row][group] replace them.  Ends with a consumer barrier.
template <typename T, int kPer>
__device__ __forceinline__ bool matvec_rows(const Params& p, Cta& c, const Desc& d, float* act, uint32_t& ring_slot,
                                            uint32_t& ring_phase) {
    constexpr int E = Chunk<T>::kElems;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int groups = d.groups, row_bytes = d.row_bytes, per_stage = d.per_stage, rows = d.a1 - d.a0;
    const int cg = warp & (groups - 1), nrg = kConsumerWarps / groups, rg = warp / groups;
    const int chunks = row_bytes / 16, S = p.stages;
    float a[kPer * E];
    uint32_t off[kPer];
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const int ch = (k * groups + cg) * 32 + lane;
        off[k] = ch < chunks ? (uint32_t)ch * 16u : 0u;
#pragma unroll
        for (int e = 0; e < E; e += 4) {
            const float4 f = ch < chunks ? *reinterpret_cast<const float4*>(act + ch * E + e) : make_float4(0.f, 0.f, 0.f, 0.f);
            a[k * E + e] = f.x;
            a[k * E + e + 1] = f.y;
            a[k * E + e + 2] = f.z;
            a[k * E + e + 3] = f.w;
        }
    }
    csync();  // everybody holds its activations: the buffer takes the partial sums
    uint32_t slot = ring_slot, phase = ring_phase;
    bool ok = true;
    for (int r0 = 0; r0 < rows; r0 += per_stage) {
        const int n = min(per_stage, rows - r0);
        const bool mine = bar_wait(p, c, c.full(slot), phase, 1);
        if (!__all_sync(0xffffffffu, mine)) {
            ok = false;
            break;
        }
        const uint32_t stage = c.base + slot * kStage;
        for (int r = rg; r < n; r += 4 * nrg) {
            float v[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int row = min(r + j * nrg, n - 1);  // (a repeated row's sum is dropped below)
                const uint32_t addr = stage + (uint32_t)row * (uint32_t)row_bytes;
                v[j] = 0.f;
#pragma unroll
                for (int k = 0; k < kPer; ++k) v[j] = Chunk<T>::dot(lds_v4(addr + off[k]), a + k * E, v[j]);
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
            if ((lane & 7) == 0 && row < n) act[(r0 + row) * groups + cg] = y;
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(c.empty(slot));
        if (++slot == (uint32_t)S) {
            slot = 0;
            phase ^= 1u;
        }
    }
    ring_slot = slot;
    ring_phase = phase;
    if (!ok) c.ctl[0] = 1;
    csync();
    return agree(c);
}

// Totals over the consumers; `red` alternates between two buffers, so that one barrier suffices.
template <int N>
__device__ __forceinline__ void csum(float* red, int& turn, float (&v)[N]) {
    float* r = red + (turn & 1) * 3 * kConsumerWarps;
    ++turn;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
    for (int n = 0; n < N; ++n) {
        v[n] = warp_sum(v[n]);
        if (lane == 0) r[n * kConsumerWarps + warp] = v[n];
    }
    csync();
#pragma unroll
    for (int n = 0; n < N; ++n) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < kConsumerWarps; w += 4) {
            const float4 f = *reinterpret_cast<const float4*>(r + n * kConsumerWarps + w);
            s += (f.x + f.y) + (f.z + f.w);
        }
        v[n] = s;
    }
}

// A vector of K floats spread over the consumers, kSlots per thread: four neighbours at a time
// where K allows 16-byte accesses, else one by one.
template <int kSlots>
struct Spread {
    float v[kSlots];
    bool wide;
    int K;
    __device__ __forceinline__ int index(int s) const {
        return wide ? 4 * ((int)threadIdx.x + kConsumers * (s >> 2)) + (s & 3) : (int)threadIdx.x + kConsumers * s;
    }
    __device__ __forceinline__ bool has(int s) const { return index(s) < K; }
    __device__ __forceinline__ void load_cg(const float* src) {
        if (wide) {
#pragma unroll
            for (int s = 0; s < kSlots; s += 4) {
                uint4 u = make_uint4(0, 0, 0, 0);
                if (has(s)) u = mkb::ld_cg_v4(src + index(s));
                v[s] = __uint_as_float(u.x);
                v[s + 1] = __uint_as_float(u.y);
                v[s + 2] = __uint_as_float(u.z);
                v[s + 3] = __uint_as_float(u.w);
            }
        } else {
#pragma unroll
            for (int s = 0; s < kSlots; ++s) v[s] = has(s) ? ld_cg_f32(src + index(s)) : 0.f;
        }
    }
    __device__ __forceinline__ void store(float* dst) const {
        if (wide) {
#pragma unroll
            for (int s = 0; s < kSlots; s += 4)
                if (has(s)) *reinterpret_cast<float4*>(dst + index(s)) = make_float4(v[s], v[s + 1], v[s + 2], v[s + 3]);
        } else {
#pragma unroll
            for (int s = 0; s < kSlots; ++s)
                if (has(s)) dst[index(s)] = v[s];
        }
        const int z = K + (int)threadIdx.x;  // padding columns
        if (z < pad8(K)) dst[z] = 0.f;
    }
};

__device__ __forceinline__ int token_id(const MkbhGlobals& g) {
    const int tok = __ldg(g.tokens);
    return tok < 0 ? 0 : tok >= g.vocab ? g.vocab - 1 : tok;
}

// Norm of the residual stream `src` (NULL: of the token's embedding, which goes to `publish` as
// well).  `part`: what earlier inputs add through the input convolution; `stash` receives the
// unweighted channels [c0, c1) for it.
template <typename T, int F, int kSlots>
__device__ __forceinline__ void norm_activation(const Params& p, const Cta& c, const float* src, const float* w, const float* part,
                                                float* act, float* red, int& turn, float* publish, float* stash, int c0, int c1) {
    const MkbhGlobals& g = p.g;
    Spread<kSlots> x;
    x.K = g.width;
    x.wide = g.width % 4 == 0;
    if (src == nullptr) {
        const T* e = static_cast<const T*>(g.embed) + (size_t)token_id(g) * x.K;
        const T* q = g.pos != nullptr ? static_cast<const T*>(g.pos) + (size_t)c.pos * x.K : nullptr;
#pragma unroll
        for (int s = 0; s < kSlots; ++s) {
            const int i = x.index(s);
            x.v[s] = i < x.K ? to_f(e[i]) * g.embed_scale + (q != nullptr ? to_f(q[i]) : 0.f) : 0.f;
            if (publish != nullptr && i < x.K) publish[i] = x.v[s];
        }
    } else {
        x.load_cg(src);
    }
    float sum[1] = {0.f};
    if (F == kClassic || ((F & kClassic) && g.norm_kind == MKBH_LAYER_NORM)) {
#pragma unroll
        for (int s = 0; s < kSlots; ++s) sum[0] += x.v[s];
        csum<1>(red, turn, sum);
        const float mean = sum[0] / x.K;
#pragma unroll
        for (int s = 0; s < kSlots; ++s) x.v[s] = x.has(s) ? x.v[s] - mean : 0.f;
    }
    sum[0] = 0.f;
#pragma unroll
    for (int s = 0; s < kSlots; ++s) sum[0] = fmaf(x.v[s], x.v[s], sum[0]);
    csum<1>(red, turn, sum);
    const float inv = 1.f / sqrtf(sum[0] / x.K + g.eps);
#pragma unroll
    for (int s = 0; s < kSlots; ++s)
        if (x.has(s)) {
            const int i = x.index(s);
            x.v[s] *= inv;
            if ((F & kRotary) && i >= c0 && i < c1) stash[i - c0] = x.v[s];
            x.v[s] = (F & kRotary) && part != nullptr ? fmaf(x.v[s], w[i], part[i]) : x.v[s] * w[i];
        }
    x.store(act);
}

// The residual stream next to the token's embedding.
template <typename T>
__device__ __forceinline__ void enter_activation(const MkbhGlobals& g, const float* src, float* act) {
    const int W = g.width;
    const T* e = static_cast<const T*>(g.embed) + (size_t)token_id(g) * W;
#pragma unroll 4
    for (int i = threadIdx.x; i < W; i += kConsumers) {
        const float x0 = to_f(e[i]) * g.embed_scale;
        act[i] = src != nullptr ? ld_cg_f32(src + i) : x0;
        act[W + i] = x0;
    }
    const int z = 2 * W + (int)threadIdx.x;
    if (z < pad8(2 * W)) act[z] = 0.f;
}

template <int kSlots>
__device__ __forceinline__ void poly_activation(const Params& p, const MkbhLayer& L, float* act, float* red, int& turn) {
    Spread<kSlots> z;
    z.K = L.ff;
    z.wide = L.ff % 4 == 0;
    z.load_cg(p.g.proj);
    float s[3] = {0.f, 0.f, 0.f};
#pragma unroll
    for (int k = 0; k < kSlots; ++k) {
        const float a = z.v[k] * z.v[k];
        s[0] += a;
        s[1] = fmaf(a, a, s[1]);
        s[2] = fmaf(a * a, a, s[2]);
    }
    csum<3>(red, turn, s);
    const float f1 = L.act[0] / sqrtf(s[0] / z.K + p.g.eps), f2 = L.act[1] / sqrtf(s[1] / z.K + p.g.eps),
                f3 = L.act[2] / sqrtf(s[2] / z.K + p.g.eps), e = L.act[3];
#pragma unroll
    for (int k = 0; k < kSlots; ++k) z.v[k] = z.v[k] * (f1 + z.v[k] * (f2 + z.v[k] * f3)) + e;
    z.store(act);
}

// Mixer output as the output projection reads it.
template <int kSlots>
__device__ __forceinline__ void plain_activation(const float* src, int K, float* act) {
    Spread<kSlots> v;
    v.K = K;
    v.wide = K % 4 == 0 && (reinterpret_cast<uint64_t>(src) & 15) == 0;
    v.load_cg(src);
    v.store(act);
}
__device__ __forceinline__ void delta_activation(const Params& p, const MkbhLayer& L, const float* w, float* act) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, D = L.dim, HD = L.heads * D;
    const float *o = p.g.mixed, *gate = p.g.proj + 4 * HD;
    for (int h0 = warp; h0 < L.heads; h0 += 2 * kConsumerWarps) {  // two heads in flight
        float v[2][kMaxChannels], g[2][kMaxChannels], s[2] = {0.f, 0.f};
#pragma unroll
        for (int b = 0; b < 2; ++b) {
            const int h = h0 + b * kConsumerWarps;
#pragma unroll
            for (int j = 0; j < kMaxChannels; ++j) {
                const int i = lane + 32 * j;
                const bool live = h < L.heads && i < D;
                v[b][j] = live ? ld_cg_f32(o + h * D + i) : 0.f;
                g[b][j] = live ? ld_cg_f32(gate + h * D + i) : 0.f;
            }
        }
#pragma unroll
        for (int b = 0; b < 2; ++b) {
            const int h = h0 + b * kConsumerWarps;
            if (h >= L.heads) break;  // uniform over the warp
#pragma unroll
            for (int j = 0; j < kMaxChannels; ++j) s[b] = fmaf(v[b][j], v[b][j], s[b]);
            const float inv = 1.f / sqrtf(warp_sum(s[b]) / D + p.g.eps);
#pragma unroll
            for (int j = 0; j < kMaxChannels; ++j) {
                const int i = lane + 32 * j;
                if (i < D) act[h * D + i] = v[b][j] * inv * w[h * D + i] * sigmoid_f(g[b][j]);
            }
        }
    }
    const int z = HD + (int)threadIdx.x;
    if (z < pad8(HD)) act[z] = 0.f;
}

// ---- generalized delta rule: one step for a block of value columns of one head --------------- //
// The state is stored column by column ([head][value column][key channel]): a warp carries one
// column, lane l the channels l, l + 32, ...; both sums over the old state (for the removal and for
// the output) are taken in one pass.
struct StateCol {
    float S[kMaxChannels];
    __device__ __forceinline__ void load(const float* col, int D, bool live) {
        const int lane = threadIdx.x & 31;
#pragma unroll
        for (int j = 0; j < kMaxChannels; ++j) S[j] = live && lane + 32 * j < D ? col[lane + 32 * j] : 0.f;
    }
};

template <typename T>
__device__ __forceinline__ void delta_step(const Params& p, const Cta& c, const Desc& d, float* act, const uint8_t* vec,
                                           const float* w0, StateCol& first) {
    const MkbhGlobals& g = p.g;
    const MkbhLayer& L = d.L;
    const int D = L.dim, HD = L.heads * D, R = L.rank, head = d.a0, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float *inner = act, *decay = act + ((R + 3) & ~3);
    const T* w2 = reinterpret_cast<const T*>(vec);
    float k[kMaxChannels], r[kMaxChannels], a[kMaxChannels];
    const float* src = g.proj + head * D;
#pragma unroll
    for (int j = 0; j < kMaxChannels; ++j) {
        const int i = lane + 32 * j;
        const bool live = i < D;
        r[j] = live ? ld_cg_f32(src + i) : 0.f;
        k[j] = live ? ld_cg_f32(src + HD + i) : 0.f;
        a[j] = live ? ld_cg_f32(src + 3 * HD + i) : 0.f;
    }
    float v = d.a1 + warp < d.a2 ? ld_cg_f32(src + 2 * HD + d.a1 + warp) : 0.f;
    for (int i = tid; i < R; i += kConsumers) inner[i] = tanhf(ld_cg_f32(g.proj + 5 * HD + i));
    // |k|^2, r . (a k), r . k
    float kk = 0.f, rak = 0.f, rk = 0.f;
#pragma unroll
    for (int j = 0; j < kMaxChannels; ++j) {
        const float x = r[j] * k[j];
        a[j] = sigmoid_f(a[j]);
        kk = fmaf(k[j], k[j], kk);
        rk += x;
        rak = fmaf(x, a[j], rak);
    }
    kk = warp_sum(kk);
    rk = warp_sum(rk);
    rak = warp_sum(rak);
    const float inv = 1.f / (kk + L.unit_eps);
    csync();
    // decays: four threads per channel, their turns skewed over the banks
    for (int i0 = 0; i0 < D; i0 += kConsumers / 4) {
        const int i = i0 + (tid >> 2);
        float s = 0.f;
        if (i < D) {
            int q = ((tid & 3) + 4 * i) % R;
            for (int n = tid & 3; n < R; n += 4) {
                s = fmaf(to_f(w2[i * R + q]), inner[q], s);
                q += 4;
                if (q >= R) q -= R;
            }
        }
        s += __shfl_xor_sync(0xffffffffu, s, 1);
        s += __shfl_xor_sync(0xffffffffu, s, 2);
        if (i < D && (tid & 3) == 0) decay[i] = expf(-L.decay_scale * sigmoid_f(s + w0[i]));
    }
    csync();
    float w[kMaxChannels];
#pragma unroll
    for (int j = 0; j < kMaxChannels; ++j) w[j] = lane + 32 * j < D ? decay[lane + 32 * j] : 0.f;
    for (int col = d.a1 + warp; col < d.a2; col += kConsumerWarps) {  // uniform over the warp
        float* S0 = L.state + (((size_t)g.slot * L.heads + head) * D + col) * D;
        if (col != d.a1 + warp) {
            first.load(S0, D, c.pos > 0);
            v = ld_cg_f32(src + 2 * HD + col);
        }
        float q = 0.f, o = 0.f;
#pragma unroll
        for (int j = 0; j < kMaxChannels; ++j) {
            q = fmaf(k[j], first.S[j], q);
            o = fmaf(r[j] * w[j], first.S[j], o);
        }
        q = warp_sum(q);
        o = warp_sum(o);
        if (lane == 0) g.mixed[head * D + col] = o - rak * inv * q + rk * v;
#pragma unroll
        for (int j = 0; j < kMaxChannels; ++j)
            if (lane + 32 * j < D) S0[lane + 32 * j] = fmaf(k[j], v - a[j] * inv * q, w[j] * first.S[j]);
    }
}

// ---- attention: one split of the keys of one KV head ----------------------------------------- //
// `maps` query vectors per head against as many keys per position (differential: 2).  Latent
// attention is one key per position, the latent with its rotated part, whose first `rank` entries
// are the value too; a "KV head" is then a group of heads.
__host__ __device__ inline int attn_maps(const MkbhLayer& L) { return L.mixer == MKBH_DIFF_ATTENTION ? 2 : 1; }
__host__ __device__ inline int attn_dim(const MkbhLayer& L) { return L.mixer == MKBH_LATENT_ATTENTION ? latent_dim(L) : L.dim; }
__host__ __device__ inline int attn_vdim(const MkbhLayer& L) { return L.mixer == MKBH_LATENT_ATTENTION ? L.rank : L.vdim; }
// Partial rows of the splits: [m, l, -, -, sums ...], 16-byte aligned.
constexpr int kPartLead = 4;
__host__ __device__ inline int part_row(int vdim) { return ((vdim + 3) & ~3) + kPartLead; }
struct AttnScratch {  // float offsets; the key and value tiles follow
    int q, p, m, l, f, own, tile;
    __host__ __device__ AttnScratch(const MkbhLayer& L, int chunk) {
        const int nq = attn_maps(L) * (L.heads / L.kv_heads), dim = attn_dim(L);
        q = 0;
        p = nq * dim;
        p = (p + 3) & ~3;
        m = p + nq * chunk;
        l = m + nq;
        f = l + nq;
        own = (f + nq + 3) & ~3;  // this token's key and value as floats
        tile = own + (L.mixer == MKBH_DIFF_ATTENTION ? 0 : (dim + attn_vdim(L) + 3) & ~3);
    }
};
template <typename T>
__host__ __device__ inline int key_stride(int elems) {  // bytes; an odd number of 16-byte units
    const int u = (elems * (int)sizeof(T) + 15) / 16;
    return (u | 1) * 16;
}
template <typename T>
__host__ __device__ inline int attn_scratch_bytes(const MkbhLayer& L, int chunk) {
    const int value = L.mixer == MKBH_LATENT_ATTENTION ? 0 : L.vdim * (int)sizeof(T);
    return AttnScratch(L, chunk).tile * 4 + chunk * (key_stride<T>(attn_maps(L) * attn_dim(L)) + value) + 16;
}
__host__ __device__ inline int merge_scratch_floats(int nq, int splits, int per, int vdim) {
    return nq * splits + per * (vdim + 1);
}

// Tensor-core variant of the one-map mixers (bf16): what it keeps in shared memory, in floats.
constexpr int kMmaKeys = 256;  // keys per pass
constexpr int kMmaCols = kMmaKeys + 8;  // scores of a head
template <typename T>
__host__ __device__ inline bool mma_attention(const MkbhLayer& L) {
    return sizeof(T) == 2 && (L.mixer == MKBH_ATTENTION || L.mixer == MKBH_LATENT_ATTENTION) && attn_dim(L) % 8 == 0 &&
           attn_vdim(L) % 8 == 0 && L.heads / L.kv_heads <= 16 && L.keep_first == 0;
}
struct MmaScratch {
    int blocks, planes, frag, p, m, l, f, own, row, krows, vrows, red, slices, groups, total;
    __host__ __device__ MmaScratch(const MkbhLayer& L) {
        const int nq = L.heads / L.kv_heads, dim = attn_dim(L), e = attn_vdim(L);
        slices = (e + 31) / 32;             // of the value columns, a warp each ...
        groups = kConsumerWarps / slices;   // ... times groups of keys
        planes = nq > 8 ? 2 : 1;
        blocks = (dim + 31) / 32;
        frag = 0;                           // queries as fragments: [plane][block][half][lane][high 2, low 2]
        p = planes * blocks * 2 * 32 * 4;
        m = p + nq * kMmaCols;
        l = m + nq;
        f = l + nq;
        own = (f + nq + 3) & ~3;            // this token's key and value: as floats ...
        row = own + ((dim + e + 3) & ~3);   // ... and as rows of bf16
        krows = row + ((dim + e + 7) / 8 * 4);  // where a pass's keys and values lie
        vrows = krows + kMmaKeys;
        red = vrows + kMmaKeys;
        total = red + (groups > 1 ? groups * nq * e : 0);
    }
};

template <typename T, int F>
struct AttnView {
    int D, KE, E, G, per, nq, ks, vs, per_stage, t_lo, count, keep, ring, pos;
    int krow, vrow;  // elements between positions
    KeyRange keys;
    T *kc, *vc, *kt, *vt;
    float *q, *p, *m, *l, *f, *own;
    bool latent, diff;
    __device__ __forceinline__ AttnView(const Params& pr, int at, const MkbhLayer& L, int kvh, int split, int splits, float* act)
        : keys(at, L.window, L.keep_first, L.chunk) {
        latent = (F & kRotary) && L.mixer == MKBH_LATENT_ATTENTION;
        diff = F == kClassic || ((F & kClassic) && L.mixer == MKBH_DIFF_ATTENTION);
        D = latent ? latent_dim(L) : L.dim; KE = diff ? 2 * D : D; E = latent ? L.rank : L.vdim;
        G = L.kv_heads; per = L.heads / G; nq = diff ? 2 * per : per;
        keep = L.cache_keep; ring = L.cache_ring; pos = at;
        const AttnScratch a(L, pr.attn_chunk);
        q = act + a.q; p = act + a.p; m = act + a.m; l = act + a.l; f = act + a.f; own = act + a.own;
        if ((F & kRotary) && mma_attention<T>(L)) {
            const MmaScratch b(L);
            p = act + b.p; m = act + b.m; l = act + b.l; f = act + b.f; own = act + b.own;
        }
        kt = reinterpret_cast<T*>(act + a.tile);
        ks = key_stride<T>(KE) / (int)sizeof(T);
        vt = latent ? kt : kt + (size_t)pr.attn_chunk * ks;
        vs = latent ? ks : E;
        per_stage = 0;
        if ((F & kRotary) && mma_attention<T>(L)) {
            ks = latent ? latent_row(L) : D;
            vs = latent ? ks : E;
            per_stage = min(kMmaKeys - 8, kStage / ((ks + (latent ? 0 : vs)) * (int)sizeof(T)));
        }
        t_lo = (int)((long long)keys.count * split / splits);
        count = (int)((long long)keys.count * (split + 1) / splits) - t_lo;
        const size_t rows0 = (size_t)pr.g.slot * (keep + ring);
        // (rotary attention keeps a KV head's rows together, differential attention a position's)
        const size_t head = diff ? kvh : ((size_t)kvh * (keep + ring));
        krow = latent ? latent_row(L) : diff ? G * KE : KE;
        vrow = diff ? G * E : E;
        kc = static_cast<T*>(L.k_cache) + (latent ? rows0 * krow : rows0 * G * KE + head * KE);
        vc = latent ? nullptr : static_cast<T*>(L.v_cache) + rows0 * G * E + head * E;
    }
    // Bring the position's rotations into L2 (they do not depend on this step).
    __device__ __forceinline__ void prefetch(const MkbhLayer& L) const {
        auto line = [](const void* a) { asm volatile("prefetch.global.L2 [%0];" ::"l"(a)); };
        const int i = threadIdx.x * 32;
        if (i < L.rope_dims) line(L.rope + (size_t)pos * L.rope_dims + i);
        if (L.value_rope != nullptr && i < L.vdim) line(L.value_rope + (size_t)pos * L.vdim + i);
    }
    __device__ __forceinline__ bool has_own() const { return count > 0 && t_lo + count == keys.count; }
    // Start copying rows [c0, c0 + nk) of the split, except this token's own: older rows do not
    // depend on this step (other layers' caches included).  One warp per key.
    __device__ __forceinline__ void stage(int c0, int nk) const {
        const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
        const int VE = latent ? 0 : E;
        const bool wide = (KE * sizeof(T)) % 16 == 0 && (VE * sizeof(T)) % 16 == 0;
        for (int t = warp; t < nk; t += kConsumerWarps) {
            const int j = keys.key(t_lo + c0 + t);
            if (j == pos) continue;
            const size_t row = cache_row(j, keep, ring);
            const T *ksrc = kc + row * krow, *vsrc = vc + row * vrow;
            T *kd = kt + t * ks, *vd = vt + t * vs;
            if (wide) {
                const int U = 16 / (int)sizeof(T), kn = KE / U, n = kn + VE / U;
                for (int u = lane; u < n; u += 32) {
                    const void* s = u < kn ? (const void*)(ksrc + u * U) : (const void*)(vsrc + (u - kn) * U);
                    const uint32_t dst = u < kn ? smem_u32(kd + u * U) : smem_u32(vd + (u - kn) * U);
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(s) : "memory");
                }
            } else {
                for (int u = lane; u < KE; u += 32) kd[u] = __ldcg(ksrc + u);
                for (int u = lane; u < VE; u += 32) vd[u] = __ldcg(vsrc + u);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
};

// ---- loader: weights, and the key/value rows of attention on tensor cores ---------------------- //
// A key/value stage holds rows as they lie in the cache: keys, then values (none for latents).
// Weights only, by one thread: a flat sequence of stages.
template <typename T>
__device__ __forceinline__ void weight_loader(const Params& p, Cta& c) {
    const MkbhGlobals& g = p.g;
    const int* queue = g.instructions + (size_t)blockIdx.x * g.queue_len * MKBH_INTS_PER_INSTRUCTION;
    const uint64_t policy = mkb::l2_policy_evict_first();
    Cursor<T> cur;
    uint32_t issued = 0;
    const uint8_t* src;
    uint32_t bytes;
    const int S = p.stages;
    while (cur.next(g, queue, src, bytes)) {
        const int slot = issued % S;
        if (!bar_wait(p, c, c.empty(slot), ((issued / S) & 1u) ^ 1u, 0)) break;
        mbar_expect_tx(c.full(slot), bytes);
        mkb::tma_bulk_g2s(c.base + slot * kStage, src, bytes, c.full(slot), policy);
        ++issued;
    }
    // no copy may be in flight when the CTA's shared memory goes away
    for (uint32_t s = issued > (uint32_t)S ? issued - S : 0u; s < issued; ++s)
        bar_wait(p, c, c.full(s % S), (s / S) & 1u, 0, false);
}

// The whole warp reads instructions (two ahead) and their layers' descriptors (one ahead), so that no
// chain of loads stands between one instruction's copies and the next one's; lane 0 waits and copies.
template <typename T, int F>
__device__ __forceinline__ void loader_main(const Params& p, Cta& c, const Smem& sm) {
    const MkbhGlobals& g = p.g;
    const int* queue = g.instructions + (size_t)blockIdx.x * g.queue_len * MKBH_INTS_PER_INSTRUCTION;
    const uint64_t policy = mkb::l2_policy_evict_first();
    const int S = p.stages, lane = threadIdx.x & 31;
    MkbhLayer* const L = reinterpret_cast<MkbhLayer*>(c.gb + sm.layer);
    constexpr int kWords = (int)sizeof(MkbhLayer) / 8, kPer = (kWords + 31) / 32;
    auto words = [&](int i) { return lane < 5 && i < g.queue_len ? __ldg(queue + (size_t)i * MKBH_INTS_PER_INSTRUCTION + lane) : 0; };
    uint2 next[kPer];
    auto fetch = [&](int layer) {
        const uint2* src = reinterpret_cast<const uint2*>(g.layers_device + layer);
#pragma unroll
        for (int k = 0; k < kPer; ++k)
            if (lane + 32 * k < kWords) next[k] = __ldg(src + lane + 32 * k);
    };
    auto keep = [&] {
        __syncwarp();
#pragma unroll
        for (int k = 0; k < kPer; ++k)
            if (lane + 32 * k < kWords) reinterpret_cast<uint2*>(L)[lane + 32 * k] = next[k];
        __syncwarp();
    };
    uint32_t issued = 0;
    int word = words(0), ahead = words(1);
    int held = __shfl_sync(0xffffffffu, word, 1);  // layer whose descriptor is there
    fetch(held);
    keep();
    bool ok = true;
    for (int i = 0; i < g.queue_len && ok; ++i) {
        int w[5];
#pragma unroll
        for (int k = 0; k < 5; ++k) w[k] = __shfl_sync(0xffffffffu, word, k);
        const int layer = __shfl_sync(0xffffffffu, ahead, 1);
        word = ahead;
        ahead = words(i + 2);
        if (layer != held) fetch(layer);
        Block b;
        if (lane != 0 || w[0] == MKBH_OP_NOOP) {
        } else if (weight_block<T>(g, w[0], L, w[2], w[3], b)) {
            const int per = kStage / b.row_bytes;
            for (int row = b.r0; row < b.r1; row += per) {
                const int slot = issued % S;
                ok = bar_wait(p, c, c.empty(slot), ((issued / S) & 1u) ^ 1u, 0);
                if (!ok) break;
                const uint32_t bytes = (uint32_t)(min(per, b.r1 - row) * b.row_bytes);
                mbar_expect_tx(c.full(slot), bytes);
                mkb::tma_bulk_g2s(c.base + slot * kStage, b.w + (size_t)row * b.row_bytes, bytes, c.full(slot), policy);
                ++issued;
            }
        } else if constexpr (sizeof(T) == 2 && (F & kRotary)) {
            if (w[0] == MKBH_OP_ATTENTION && mma_attention<T>(*L)) {
                const AttnView<T, F> A(p, c.pos, *L, w[2], w[3], w[4], nullptr);
                const int old = A.count - (A.has_own() ? 1 : 0);
                for (int k0 = 0; k0 < old; k0 += A.per_stage) {
                    const int slot = issued % S, n = min(A.per_stage, old - k0);
                    ok = bar_wait(p, c, c.empty(slot), ((issued / S) & 1u) ^ 1u, 0);
                    if (!ok) break;
                    const uint32_t kd = c.base + slot * kStage, vd = kd + A.per_stage * A.ks * (int)sizeof(T);
                    const uint32_t kb = A.ks * (int)sizeof(T), vb = A.latent ? 0 : A.vs * (int)sizeof(T);
                    mbar_expect_tx(c.full(slot), n * (kb + vb));
                    // the rows are neighbours but where the ring ends
                    for (int t = 0; t < n;) {
                        const int row = cache_row(A.keys.key(A.t_lo + k0 + t), A.keep, A.ring), run = min(n - t, A.keep + A.ring - row);
                        mkb::tma_bulk_g2s(kd + t * kb, A.kc + (size_t)row * A.krow, run * kb, c.full(slot), policy);
                        if (vb) mkb::tma_bulk_g2s(vd + t * vb, A.vc + (size_t)row * A.vrow, run * vb, c.full(slot), policy);
                        t += run;
                    }
                    ++issued;
                }
            }
        }
        ok = __shfl_sync(0xffffffffu, ok, 0);
        if (layer != held) {
            keep();
            held = layer;
        }
    }
    if (lane != 0) return;
    // no copy may be in flight when the CTA's shared memory goes away
    for (uint32_t s = issued > (uint32_t)S ? issued - S : 0u; s < issued; ++s)
        bar_wait(p, c, c.full(s % S), (s / S) & 1u, 0, false);
}

// What an attention instruction fetches before its producers are done.
template <typename T, int F>
__device__ __forceinline__ void attend_ahead(const Params& pr, int pos, const Desc& d, float* act) {
    const AttnView<T, F> A(pr, pos, d.L, d.a0, d.a1, d.a2, act);
    if ((F & kRotary) && mma_attention<T>(d.L)) A.prefetch(d.L);
    else A.stage(0, min(pr.attn_chunk, A.count));
}

// One head's vector, by one warp: optional norm (weight w), rotation of the first `rot` elements
// (neighbours by the angles of `rope`), factor `mul`.  All of it is read before anything is used;
// n <= 64 J.
struct HeadOut {  // floats at dst, or (frag) the high and low bf16 parts in fragment order of row `head`
    float* dst;
    uint32_t* frag;
    int head, col0;
    __device__ __forceinline__ void put(int i, int n, float x, float y) const {  // columns i (even), i + 1
        if (i >= n) return;
        if (frag == nullptr) {
            dst[i] = x;
            if (i + 1 < n) dst[i + 1] = y;
            return;
        }
        const int col = col0 + i;  // (heads of an odd size have no fragments)
        uint32_t* f = frag + (((col >> 5) * 2 + (col >> 2 & 1)) * 32 + (head & 7) * 4 + (col >> 3 & 3)) * 4 + (col >> 1 & 1);
        const uint32_t hi = mkb::pack_bf16x2(x, y);
        f[0] = hi;
        f[2] = mkb::pack_bf16x2(x - mkb::bf16_lo(hi), y - mkb::bf16_hi(hi));
    }
};
template <int J>
__device__ __forceinline__ void head_vector(const float* src, int n, const float* w, float eps, const float2* rope, int rot,
                                            float mul, const HeadOut& out) {
    const int lane = threadIdx.x & 31;
    float a[J], b[J], wa[J], wb[J], s = 0.f;
    float2 r[J];
#pragma unroll
    for (int j = 0; j < J; ++j) {
        const int i = 2 * (lane + 32 * j);
        a[j] = i < n ? ld_cg_f32(src + i) : 0.f;
        b[j] = i + 1 < n ? ld_cg_f32(src + i + 1) : 0.f;
        wa[j] = w != nullptr && i < n ? __ldg(w + i) : 1.f;
        wb[j] = w != nullptr && i + 1 < n ? __ldg(w + i + 1) : 1.f;
        r[j] = i < rot ? __ldg(rope + (i >> 1)) : make_float2(1.f, 0.f);
    }
    if (w != nullptr) {
#pragma unroll
        for (int j = 0; j < J; ++j) s = fmaf(a[j], a[j], fmaf(b[j], b[j], s));
        s = 1.f / sqrtf(warp_sum(s) / n + eps);
    } else {
        s = 1.f;
    }
#pragma unroll
    for (int j = 0; j < J; ++j) {
        const int i = 2 * (lane + 32 * j);
        const float x = a[j] * s * wa[j], y = b[j] * s * wb[j];
        out.put(i, n, (x * r[j].x - y * r[j].y) * mul, (y * r[j].x + x * r[j].y) * mul);
    }
}
// (by size: one call site each for up to 64, 128 and 512 elements)
__device__ __noinline__ void head_vector_any(const float* src, int n, const float* w, float eps, const float2* rope, int rot,
                                             float mul, const HeadOut out) {
    if (n <= 64) head_vector<1>(src, n, w, eps, rope, rot, mul, out);
    else if (n <= 128) head_vector<2>(src, n, w, eps, rope, rot, mul, out);
    else head_vector<8>(src, n, w, eps, rope, rot, mul, out);
}

// Queries of the KV head's heads, normalised, rotated and scaled, and, in the split that holds it,
// this token's key and value.  Ends with a barrier.
// `frag`: where the queries go as fragments (NULL: floats at A.q).
template <typename T, int F>
__device__ __forceinline__ void rotary_operands(const Params& pr, const AttnView<T, F>& A, const MkbhLayer& L, int kvh, uint32_t* frag) {
    const MkbhGlobals& g = pr.g;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tasks = A.nq + (A.has_own() ? 2 : 0);
    const float2* rope = reinterpret_cast<const float2*>(L.rope) + (size_t)A.pos * (L.rope_dims / 2);
    for (int t = warp; t < tasks; t += kConsumerWarps) {
        const int h = kvh * A.per + t;
        const bool query = t < A.nq, first = t == A.nq;
        const float *src, *w = nullptr;
        const float2* angles = rope;
        int n, rot = L.rope_dims;
        float mul = 1.f;
        HeadOut out{query ? A.q + t * A.D : A.own, query && frag != nullptr ? frag + (t >> 3) * ((A.D + 31) / 32) * 256 : nullptr, t, 0};
        if (A.latent) {
            const int hd = L.dim + L.rot_dim, lead = pad8(L.rank);
            const float* down = g.proj + (size_t)L.heads * hd;
            if (query) {
                const float* absorbed = side_query(g) + (size_t)h * L.rank;
                mul = L.scale;
                for (int i0 = 0; i0 < lead; i0 += 512) {
                    float x[8], y[8];
#pragma unroll
                    for (int j = 0; j < 8; ++j) {
                        const int i = i0 + 2 * (lane + 32 * j);
                        x[j] = i < L.rank ? ld_cg_f32(absorbed + i) * mul : 0.f;
                        y[j] = i + 1 < L.rank ? ld_cg_f32(absorbed + i + 1) * mul : 0.f;
                    }
#pragma unroll
                    for (int j = 0; j < 8; ++j) out.put(i0 + 2 * (lane + 32 * j), lead, x[j], y[j]);
                }
            }
            if (!first) {  // rotated part
                src = query ? g.proj + (size_t)h * hd + L.dim : down + L.rank;
                n = L.rot_dim;
                if (out.frag == nullptr) out.dst += lead;
                else out.col0 = lead;
                for (int i = (n & ~1) + 2 * lane; i < A.D - lead; i += 64) out.put(i, A.D - lead, 0.f, 0.f);
            } else {
                src = down;
                n = L.rank;
                w = L.k_norm;
                rot = 0;
                for (int i = L.rank + lane; i < lead; i += 32) out.dst[i] = 0.f;
            }
            __syncwarp();
        } else if (query) {
            src = g.proj + (size_t)h * A.D;
            n = A.D;
            w = L.q_norm;
            mul = L.scale * __ldg(L.temp + h);
        } else if (first) {
            src = g.proj + (size_t)(L.heads + kvh) * A.D;
            n = A.D;
            w = L.k_norm;
        } else {
            src = g.proj + (size_t)(L.heads + A.G) * A.D + (size_t)kvh * A.E;
            n = A.E;
            angles = reinterpret_cast<const float2*>(L.value_rope) + (size_t)A.pos * (A.E / 2);
            rot = L.value_rope != nullptr ? A.E : 0;
            out.dst += A.D;
        }
        head_vector_any(src, n, w, g.eps, angles, rot, mul, out);
    }
    csync();
}

template <typename T, int F, int kAcc>
__device__ __forceinline__ void attend(const Params& pr, const AttnView<T, F>& A, const Desc& d) {
    const MkbhGlobals& g = pr.g;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, KC = pr.attn_chunk;
    const int D = A.D, E = A.E, nq = A.nq, kvh = d.a0;
    const bool diff = A.diff;
    const float scale = diff ? d.L.scale : 1.f;
    const bool owns = d.L.owns_kv != 0;
    const int kv_off = d.L.heads * (2 * D + E);
    const int lanes_e = kConsumers / E;  // query vectors served side by side (E <= 512)
    const int e = tid % E, qv0 = tid / E;
    const bool has_e = qv0 < lanes_e;
    const bool dot16 = (D * sizeof(T)) % 16 == 0;
    float acc[kAcc];
#pragma unroll
    for (int i = 0; i < kAcc; ++i) acc[i] = 0.f;
    if (diff)
        for (int i = tid; i < nq * D; i += kConsumers) A.q[i] = ld_cg_f32(g.proj + (size_t)kvh * nq * D + i);
    else if constexpr (F & kRotary)
        rotary_operands<T, F>(pr, A, d.L, kvh, nullptr);

    for (int c0 = 0; c0 < A.count; c0 += KC) {
        const int nk = min(KC, A.count - c0);
        if (c0 > 0) A.stage(c0, nk);
        if (A.keys.key(A.t_lo + c0 + nk - 1) == A.pos) {  // this token's own row (always the last key)
            const int t = nk - 1;
            const size_t row = cache_row(A.pos, A.keep, A.ring);
            const int KE = A.KE;
            for (int i = tid; i < KE + (A.latent ? 0 : E); i += kConsumers) {
                const bool is_k = i < KE;
                T* cell = is_k ? A.kc + row * A.krow + i : A.vc + row * A.vrow + (i - KE);
                T x;
                if (!diff) {
                    x = from_f<T>(A.own[i]);
                    if (!A.latent || kvh == 0) *cell = x;  // (every group of heads has the same latent)
                } else if (owns) {
                    x = from_f<T>(ld_cg_f32(g.proj + kv_off + (is_k ? kvh * KE + i : A.G * KE + kvh * E + (i - KE))));
                    *cell = x;
                } else {
                    x = __ldcg(cell);
                }
                if (is_k) A.kt[t * A.ks + i] = x;
                else A.vt[t * A.vs + (i - KE)] = x;
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        csync();
        // scores: consecutive threads take consecutive keys of one query vector
        for (int i = tid; i < nq * KC; i += kConsumers) {
            const int t = i % KC, qv = i / KC;
            float s = -INFINITY;
            if (t < nk) {
                const T* k = A.kt + t * A.ks + (diff ? (qv & 1) * D : 0);
                const float* qq = A.q + qv * D;
                s = 0.f;
                if (dot16) {
                    constexpr int U = Chunk<T>::kElems;
#pragma unroll 4
                    for (int n = 0; n < D; n += U) {
                        float f[U];
#pragma unroll
                        for (int x = 0; x < U; x += 4) {
                            const float4 y = *reinterpret_cast<const float4*>(qq + n + x);
                            f[x] = y.x; f[x + 1] = y.y; f[x + 2] = y.z; f[x + 3] = y.w;
                        }
                        s = Chunk<T>::dot(lds_v4(smem_u32(k + n)), f, s);
                    }
                } else {
                    for (int n = 0; n < D; ++n) s = fmaf(to_f(k[n]), qq[n], s);
                }
                s *= scale;
            }
            A.p[qv * KC + t] = s;
        }
        csync();
        for (int qv = warp; qv < nq; qv += kConsumerWarps) {
            const float old = c0 > 0 ? A.m[qv] : -INFINITY;
            float x = -INFINITY;
            for (int t = lane; t < KC; t += 32) x = fmaxf(x, A.p[qv * KC + t]);
            x = fmaxf(warp_max(x), old);
            float s = 0.f;
            for (int t = lane; t < KC; t += 32) {
                const float y = expf(A.p[qv * KC + t] - x);
                A.p[qv * KC + t] = y;
                s += y;
            }
            s = warp_sum(s);
            if (lane == 0) {
                const float fac = expf(old - x);
                A.l[qv] = (c0 > 0 ? A.l[qv] * fac : 0.f) + s;
                A.f[qv] = fac;
                A.m[qv] = x;
            }
        }
        csync();
        if (has_e) {
            if (c0 > 0) {
#pragma unroll
                for (int i = 0; i < kAcc; ++i)
                    if (qv0 + i * lanes_e < nq) acc[i] *= A.f[qv0 + i * lanes_e];
            }
            for (int t = 0; t < nk; t += 4) {  // weights beyond nk are zero
                float v[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) v[j] = t + j < nk ? to_f(A.vt[(t + j) * A.vs + e]) : 0.f;
#pragma unroll
                for (int i = 0; i < kAcc; ++i) {
                    const int qv = qv0 + i * lanes_e;
                    if (qv < nq) {
                        const float4 w4 = *reinterpret_cast<const float4*>(A.p + qv * KC + t);
                        acc[i] = fmaf(w4.x, v[0], fmaf(w4.y, v[1], fmaf(w4.z, v[2], fmaf(w4.w, v[3], acc[i]))));
                    }
                }
            }
        }
        csync();
    }
    // partial rows [head and map][split][m, l, acc...]
    const int PE = part_row(g.part_vdim), split = d.a1;
    float* part = g.attn_part + (size_t)kvh * nq * g.max_splits * PE;
    if (has_e) {
#pragma unroll
        for (int i = 0; i < kAcc; ++i) {
            const int qv = qv0 + i * lanes_e;
            if (qv < nq) {
                float* row = part + ((size_t)qv * g.max_splits + split) * PE;
                row[kPartLead + e] = acc[i];
                if (e == 0) {
                    row[0] = A.count > 0 ? A.m[qv] : -INFINITY;
                    row[1] = A.count > 0 ? A.l[qv] : 0.f;
                }
            }
        }
    }
}

template <typename T, int F>
__device__ __forceinline__ void attend_fma(const Params& pr, int pos, const Desc& d, float* act) {
    const AttnView<T, F> A(pr, pos, d.L, d.a0, d.a1, d.a2, act);
    const int need = (A.nq + kConsumers / A.E - 1) / (kConsumers / A.E);
    if (need <= 2) attend<T, F, 2>(pr, A, d);
    else if (need <= 4) attend<T, F, 4>(pr, A, d);
    else attend<T, F, 16>(pr, A, d);
}

__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = mkb::pack_bf16x2(x, y);
    lo = mkb::pack_bf16x2(x - mkb::bf16_lo(hi), y - mkb::bf16_hi(hi));
}

// One split on mma.sync, from the ring's key/value stages: the M side of both products are the heads of
// the group (queries and softmax weights enter as a high and a low bf16 part), the N side keys, then
// value columns.  The index of a contraction may be permuted as long as both operands agree, so a
// lane's share of a fragment is a run of neighbours in memory.
template <typename T, int F>
__device__ __forceinline__ bool attend_mma(const Params& pr, Cta& cta, const Desc& d, float* act, uint32_t& ring_slot, uint32_t& ring_phase) {
    const MkbhGlobals& g = pr.g;
    const int pos = cta.pos;
    const AttnView<T, F> A(pr, pos, d.L, d.a0, d.a1, d.a2, act);
    const MmaScratch S(d.L);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane >> 2, c = lane & 3;
    const int D = A.D, E = A.E, nq = A.nq, kvh = d.a0;
    const bool own = A.has_own(), latent = A.latent;
    float *const p = A.p, *const red = act + S.red;
    const uint4* const frag = reinterpret_cast<const uint4*>(act + S.frag);
    const int slice = warp % S.slices, group = warp / S.slices, e0 = slice * 32 + r * 4;
    int *const krows = reinterpret_cast<int*>(act + S.krows), *const vrows = reinterpret_cast<int*>(act + S.vrows);
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    // (columns beyond the heads' size and rows beyond their number are zero)
    for (int i = tid; i < S.planes * S.blocks * 64; i += kConsumers) reinterpret_cast<uint4*>(act + S.frag)[i] = make_uint4(0, 0, 0, 0);
    csync();
    rotary_operands<T, F>(pr, A, d.L, kvh, reinterpret_cast<uint32_t*>(act + S.frag));
    const int blocks = S.blocks;
    T* const own_row = reinterpret_cast<T*>(act + S.row);
    if (own) {  // this token's row
        const size_t row = cache_row(pos, A.keep, A.ring);
        for (int i = tid; i < D + (latent ? 0 : E); i += kConsumers) {
            const T x = from_f<T>(A.own[i]);
            own_row[i] = x;
            if (!latent || kvh == 0)  // (every group of heads has the same latent)
                (i < D ? A.kc[row * A.krow + i] : A.vc[row * A.vrow + (i - D)]) = x;
        }
    }
    const int old = A.count - (own ? 1 : 0), per_stage = A.per_stage;
    const int most = max(1, min(pr.stages, (kMmaKeys - 1) / per_stage)), pass = most * per_stage;  // stages, keys of a pass
    for (int c0 = 0; c0 == 0 || c0 < old; c0 += pass) {
        const int staged = min(pass, old - c0), stages = (staged + per_stage - 1) / per_stage;
        const bool last = c0 + pass >= old;
        const int n = staged + (last && own ? 1 : 0);  // this token's own key comes last
        if (c0 > 0) csync();  // the buffers are free
        if (tid == 0 && n > staged) {
            krows[staged] = (int)(smem_u32(own_row) - cta.base);
            vrows[staged] = krows[staged] + (latent ? 0 : D * (int)sizeof(T));
        }
        for (int i = tid; i < staged; i += kConsumers) {
            const int st = i / per_stage, j = i - st * per_stage, at = (int)((ring_slot + st) % pr.stages) * kStage;
            krows[i] = at + j * A.ks * (int)sizeof(T);
            vrows[i] = latent ? krows[i] : at + (per_stage * A.ks + j * A.vs) * (int)sizeof(T);
        }
        bool ok = true;
        uint32_t slot = ring_slot, phase = ring_phase;
        for (int i = 0; i < stages && ok; ++i) {
            ok = bar_wait(pr, cta, cta.full(slot), phase, 1);
            if (++slot == (uint32_t)pr.stages) slot = 0, phase ^= 1u;
        }
        if (!__all_sync(0xffffffffu, ok)) cta.ctl[0] = 1;
        if (!agree(cta)) return false;
        // scores: a warp takes tiles of 8 keys; lane (r, c) holds eight neighbours of key r's row per 32
        for (int t = warp; t * 8 < n; t += kConsumerWarps) {
            const bool live = t * 8 + r < n;
            const uint32_t k = cta.base + krows[live ? t * 8 + r : 0] + c * 16;
            float s[2][4] = {};
            for (int b0 = 0; b0 < blocks; b0 += 6) {
                uint4 kv[6];
#pragma unroll
                for (int i = 0; i < 6; ++i)
                    kv[i] = live && (b0 + i) * 32 + c * 8 < D ? lds_v4(k + (b0 + i) * 64) : make_uint4(0, 0, 0, 0);
#pragma unroll
                for (int i = 0; i < 6; ++i) {
                    if (b0 + i >= blocks) break;
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
                        const uint4 x = frag[((b0 + i) * 2 + h) * 32 + lane];
                        uint4 y = make_uint4(0, 0, 0, 0);
                        if (S.planes > 1) y = frag[((blocks + b0 + i) * 2 + h) * 32 + lane];
                        const uint32_t hi[4] = {x.x, y.x, x.y, y.y}, lo[4] = {x.z, y.z, x.w, y.w};
                        const uint32_t k0 = h ? kv[i].z : kv[i].x, k1 = h ? kv[i].w : kv[i].y;
                        mma_16816(s[0], hi, k0, k1);
                        mma_16816(s[1], lo, k0, k1);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int head = r + 8 * (j >> 1), key = t * 8 + 2 * c + (j & 1);
                if (head < nq) p[head * kMmaCols + key] = key < n ? s[0][j] + s[1][j] : -INFINITY;
            }
        }
        csync();
        const int padded = (n + 15) & ~15;
        for (int h = warp; h < nq; h += kConsumerWarps) {
            float* row = p + h * kMmaCols;
            const float before = c0 > 0 ? A.m[h] : -INFINITY;
            float v[kMmaKeys / 32], x = before;
#pragma unroll
            for (int j = 0; j < kMmaKeys / 32; ++j) {
                v[j] = lane + 32 * j < n ? row[lane + 32 * j] : -INFINITY;
                x = fmaxf(x, v[j]);
            }
            x = warp_max(x);
            float s = 0.f;
#pragma unroll
            for (int j = 0; j < kMmaKeys / 32; ++j) {
                const float y = x == -INFINITY ? 0.f : expf(v[j] - x);
                if (lane + 32 * j < padded) row[lane + 32 * j] = y;
                s += y;
            }
            s = warp_sum(s);
            if (lane == 0) {
                const float fac = x == -INFINITY ? 1.f : expf(before - x);
                A.l[h] = (c0 > 0 ? A.l[h] * fac : 0.f) + s;
                A.f[h] = fac;
                A.m[h] = x;
            }
        }
        csync();
        if (group < S.groups) {
            if (c0 > 0) {
                const float f0 = r < nq ? A.f[r] : 0.f, f1 = r + 8 < nq ? A.f[r + 8] : 0.f;
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    acc[i][0] *= f0;
                    acc[i][1] *= f0;
                    acc[i][2] *= f1;
                    acc[i][3] *= f1;
                }
            }
            // a warp takes 32 value columns and every groups-th run of 16 keys, four runs at a time
            const int step = 16 * S.groups;
            for (int k0 = group * 16; k0 < n; k0 += 4 * step) {
                uint2 v[4][4];
#pragma unroll
                for (int u = 0; u < 4; ++u)
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const int key = k0 + u * step + 2 * c + (j & 1) + 8 * (j >> 1);
                        v[u][j] = make_uint2(0, 0);
                        if (key < n && e0 < E) v[u][j] = mkb::lds_v2(cta.base + vrows[key] + e0 * 2);
                    }
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    const int k = k0 + u * step;
                    if (k >= n) break;
                    uint32_t hi[4] = {}, lo[4] = {};
                    const float* row = p + r * kMmaCols + k + 2 * c;
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        if (r + 8 * (j & 1) >= nq) continue;
                        const float2 y = *reinterpret_cast<const float2*>(row + (j & 1) * 8 * kMmaCols + 8 * (j >> 1));
                        split_bf16(y.x, y.y, hi[j], lo[j]);
                    }
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const uint32_t a0 = j < 2 ? v[u][0].x : v[u][0].y, a1 = j < 2 ? v[u][1].x : v[u][1].y;
                        const uint32_t a2 = j < 2 ? v[u][2].x : v[u][2].y, a3 = j < 2 ? v[u][3].x : v[u][3].y;
                        const uint32_t sel = j & 1 ? 0x7632u : 0x5410u, b0 = __byte_perm(a0, a1, sel), b1 = __byte_perm(a2, a3, sel);
                        mma_16816(acc[j], hi, b0, b1);
                        mma_16816(acc[j], lo, b0, b1);
                    }
                }
            }
        }
        __syncwarp();
        for (int i = 0; i < stages; ++i) {
            if (lane == 0) mbar_arrive(cta.empty(ring_slot));
            if (++ring_slot == (uint32_t)pr.stages) ring_slot = 0, ring_phase ^= 1u;
        }
    }
    // this lane's sums: heads r and r + 8, four neighbouring columns for each of two indices
    const int PE = part_row(g.part_vdim), max_splits = g.max_splits;
    float* const part = g.attn_part + ((size_t)kvh * nq * max_splits + d.a1) * PE;
    auto out = [&](float* dst, size_t ld) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int head = r + 8 * (j >> 1), e = slice * 32 + (2 * c + (j & 1)) * 4;
            if (head < nq && e < E)  // (E is a multiple of 8)
                *reinterpret_cast<float4*>(dst + head * ld + e) = make_float4(acc[0][j], acc[1][j], acc[2][j], acc[3][j]);
        }
    };
    if (S.groups == 1) {
        if (group == 0) out(part + kPartLead, (size_t)max_splits * PE);
    } else {
        if (group < S.groups) out(red + group * nq * E, E);
        csync();
        for (int i = tid; i < nq * E; i += kConsumers) {
            const int h = i / E, e = i - h * E;
            float y = 0.f;
            for (int k = 0; k < S.groups; ++k) y += red[k * nq * E + i];
            part[(size_t)h * max_splits * PE + kPartLead + e] = y;
        }
    }
    if (tid < nq) {
        part[(size_t)tid * max_splits * PE] = A.m[tid];
        part[(size_t)tid * max_splits * PE + 1] = A.l[tid];
    }
    return true;
}

// Output of a latent attention's head in latent space, merged over the splits: the input of its
// expansion.  Every warp works out the splits' factors while the partial rows are on their way; a
// quarter of the threads takes every fourth split.
__device__ __forceinline__ void latent_activation(const Params& pr, const MkbhLayer& L, int head, int splits, float* act) {
    const MkbhGlobals& g = pr.g;
    const int lane = threadIdx.x & 31, PE = part_row(g.part_vdim), e = 4 * (threadIdx.x & 127), quarter = threadIdx.x >> 7, rank = L.rank;
    const float* row = g.attn_part + (size_t)head * g.max_splits * PE;
    float m[2], l[2], f[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const bool live = lane + 32 * h < splits;
        m[h] = live ? ld_cg_f32(row + (size_t)(lane + 32 * h) * PE) : -INFINITY;
        l[h] = live ? ld_cg_f32(row + (size_t)(lane + 32 * h) * PE + 1) : 0.f;
    }
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s0 = quarter; s0 < splits; s0 += 32) {
        uint4 x[8];
#pragma unroll
        for (int j = 0; j < 8; ++j)
            x[j] = e < rank && s0 + 4 * j < splits ? mkb::ld_cg_v4(row + (size_t)(s0 + 4 * j) * PE + kPartLead + e) : make_uint4(0, 0, 0, 0);
        if (s0 == quarter) {
            const float top = warp_max(fmaxf(m[0], m[1]));
            f[0] = expf(m[0] - top);
            f[1] = expf(m[1] - top);
            const float inv = 1.f / warp_sum(l[0] * f[0] + l[1] * f[1]);
            f[0] *= inv;
            f[1] *= inv;
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int s = s0 + 4 * j;  // (uniform over the warp)
            const float w = __shfl_sync(0xffffffffu, s & 32 ? f[1] : f[0], s & 31);
            y.x = fmaf(w, __uint_as_float(x[j].x), y.x);
            y.y = fmaf(w, __uint_as_float(x[j].y), y.y);
            y.z = fmaf(w, __uint_as_float(x[j].z), y.z);
            y.w = fmaf(w, __uint_as_float(x[j].w), y.w);
        }
    }
    float* red = act + 512;
    *reinterpret_cast<float4*>(red + quarter * 512 + e) = y;
    csync();
    const int i = threadIdx.x;
    if (i < pad8(rank)) act[i] = i < rank ? (red[i] + red[512 + i]) + (red[1024 + i] + red[1536 + i]) : 0.f;
}

// The split of a KV head that arrives last merges the partial rows.  Differential: combines the
// maps, normalises and gates.  Rotary: turns the outputs back.
template <bool kDiff>
__device__ __forceinline__ void merge_splits(const Params& pr, int pos, const Desc& d, float* act) {
    const MkbhGlobals& g = pr.g;
    const MkbhLayer& L = d.L;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, max_splits = g.max_splits;
    const int E = L.vdim, per = L.heads / L.kv_heads, maps = kDiff ? 2 : 1, nq = maps * per, kvh = d.a0, splits = d.a2, PE = part_row(g.part_vdim);
    const float* part = g.attn_part + (size_t)kvh * nq * max_splits * PE;
    float *fac = act, *o = act + nq * splits, *norm = o + per * E;
    for (int qv = warp; qv < nq; qv += kConsumerWarps) {
        const float* row = part + ((size_t)qv * max_splits + lane) * PE;
        const float m = lane < splits ? ld_cg_f32(row) : -INFINITY, l = lane < splits ? ld_cg_f32(row + 1) : 0.f;
        const float sink = !kDiff && L.sink != nullptr ? __ldg(L.sink + kvh * per + qv) : -INFINITY;
        const float top = fmaxf(warp_max(m), sink), f = expf(m - top), total = warp_sum(l * f) + (kDiff ? 0.f : expf(sink - top));
        if (lane < splits) fac[qv * splits + lane] = f / total;
    }
    csync();
    for (int i = tid; i < per * E; i += kConsumers) {
        const int hh = i / E, e = i % E;
        const float *s1 = part + (size_t)(maps * hh) * max_splits * PE + kPartLead + e, *s2 = s1 + (size_t)max_splits * PE;
        const float *f1 = fac + maps * hh * splits, *f2 = f1 + splits;
        constexpr int B = kDiff ? 8 : 16;  // splits in flight
        float a1 = 0.f, a2 = 0.f;
        for (int s = 0; s < splits; s += B) {
            float x[B], y[B];
#pragma unroll
            for (int j = 0; j < B; ++j) {
                x[j] = s + j < splits ? ld_cg_f32(s1 + (size_t)(s + j) * PE) : 0.f;
                if constexpr (kDiff) y[j] = s + j < splits ? ld_cg_f32(s2 + (size_t)(s + j) * PE) : 0.f;
            }
#pragma unroll
            for (int j = 0; j < B; ++j)
                if (s + j < splits) {
                    a1 = fmaf(f1[s + j], x[j], a1);
                    if constexpr (kDiff) a2 = fmaf(f2[s + j], y[j], a2);
                }
        }
        o[i] = kDiff ? a1 - L.lambda * a2 : a1;
    }
    csync();
    if constexpr (!kDiff) {
        const float2* turn = L.value_rope == nullptr ? nullptr : reinterpret_cast<const float2*>(L.value_rope) + (size_t)pos * (E / 2);
        for (int i = tid; i < per * E; i += kConsumers) {
            float y = o[i];
            if (turn != nullptr) {  // (an even number of elements per head)
                const float2 r = __ldg(turn + (i % E >> 1));
                y = y * r.x + (i & 1 ? -r.y : r.y) * o[i ^ 1];
            }
            g.mixed[(size_t)kvh * per * E + i] = y;
        }
    } else {
        for (int hh = warp; hh < per; hh += kConsumerWarps) {
            float s = 0.f;
            for (int e = lane; e < E; e += 32) s = fmaf(o[hh * E + e], o[hh * E + e], s);
            s = warp_sum(s);
            if (lane == 0) norm[hh] = (1.f - L.diff) / sqrtf(s / E + g.eps);
        }
        csync();
        const float* gate = g.proj + L.heads * 2 * L.dim + (size_t)kvh * per * E;
        for (int i = tid; i < per * E; i += kConsumers)
            g.mixed[(size_t)kvh * per * E + i] = o[i] * norm[i / E] * sigmoid_f(ld_cg_f32(gate + i));
    }
}

// Short convolutions over time: keep this token's inputs and sum up the terms of the next token's
// earlier inputs.  `stash` holds the normalised channels of the instruction's share of the mixer's
// input, `u` is this thread's row of the stacked projection before its convolution.
__device__ __forceinline__ void keep_input(float now, const float* w, float* hist, float* next, int taps, size_t ld, int pos) {
    float s = __ldg(w + (taps - 2) * ld) * now;
    for (int i0 = 1; i0 <= taps - 2; i0 += 4) {
        float a[4], b[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = i0 + j;
            const bool live = i <= taps - 2 && i <= pos;
            a[j] = live ? __ldg(w + (taps - 2 - i) * ld) : 0.f;
            b[j] = live ? hist[((pos - i) % (taps - 1)) * ld] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) s = fmaf(a[j], b[j], s);
    }
    hist[(pos % (taps - 1)) * ld] = now;
    *next = s;
}
__device__ __forceinline__ void publish_convolutions(const Params& p, const Cta& c, const Desc& d, const float* stash, float u) {
    const MkbhGlobals& g = p.g;
    const MkbhLayer& L = d.L;
    const int tid = threadIdx.x, lo = (int)((long long)g.width * d.a0 / L.in_rows), hi = (int)((long long)g.width * d.a1 / L.in_rows);
    if (L.canon_taps > 1 && tid < hi - lo) {
        const int ch = lo + tid;
        keep_input(stash[tid] * __ldg(L.norm1 + ch), L.canon_w + ch,
                   L.canon_hist + (size_t)g.slot * (L.canon_taps - 1) * g.width + ch,
                   L.canon_part + ((size_t)g.slot * 2 + ((c.pos + 1) & 1)) * g.width + ch, L.canon_taps, g.width, c.pos);
    }
    if (L.conv_taps > 1 && tid < d.a1 - d.a0) {
        const int row = d.a0 + tid;
        keep_input(u, L.conv_w + row, L.conv_hist + (size_t)g.slot * (L.conv_taps - 1) * L.in_rows + row,
                   L.conv_part + (size_t)g.slot * L.in_rows + row, L.conv_taps, L.in_rows, c.pos);
    }
}

__device__ __forceinline__ unsigned long long argmax_key(float v, int i) {
    uint32_t u = __float_as_uint(v);
    u = (u >> 31) ? ~u : (u | 0x80000000u);
    return ((unsigned long long)u << 32) | (0xffffffffu - (uint32_t)i);
}

template <typename T, int F>
__device__ __forceinline__ void consumer_main(const Params& p, Cta& c, const Smem& sm) {
    const MkbhGlobals& g = p.g;
    const int tid = threadIdx.x, warp = tid >> 5;
    float* act = reinterpret_cast<float*>(c.gb + sm.act);
    float* red = reinterpret_cast<float*>(c.gb + sm.red);
    float* stash = reinterpret_cast<float*>(c.gb + sm.stash);
    int* counters = g.counters + 2;
    uint32_t slot = 0, phase = 0, vecs = 0;
    int turn = 0;
    for (int i = 0; i < g.queue_len; ++i) {
        c.instr = i;
        c.opcode = -1;
        bool ok = bar_wait(p, c, c.bar(kDescFull + (i & 1)), (i >> 1) & 1u, 1);
        if (!ok) c.ctl[0] = 1;
        if (!agree(c)) return;  // (a barrier per instruction; it also separates the scratch's users)
        const Desc& d = *reinterpret_cast<const Desc*>(c.gb + sm.desc + (i & 1) * kDescBytes);
        const MkbhLayer& L = d.L;
        const float* rowv = reinterpret_cast<const float*>(c.gb + sm.rows + (i & 1) * kRowVecBytes + max(d.row_off, 0));
        const uint8_t* vec = c.gb + sm.vec + d.vec_off;
        const int op = c.opcode = d.op;
        int* stamp = g.timings != nullptr && tid == 0 ? g.timings + ((size_t)blockIdx.x * g.queue_len + i) * MKBH_TIMING_SLOTS : nullptr;
        auto rec = [&](int k) {
            if (stamp) stamp[k] = (int)(uint32_t)globaltimer_ns();
        };
        if (op == MKBH_OP_NOOP) {
            csync();
            if (tid == 0) mbar_arrive(c.bar(kDescEmpty + (i & 1)));
            continue;
        }
        rec(0);
        // ---- what does not depend on the producers ----
        StateCol state;
        if ((F & kClassic) && op == MKBH_OP_DELTA_STEP)
            state.load(L.state + (((size_t)g.slot * L.heads + d.a0) * L.dim + d.a1 + warp) * L.dim, L.dim,
                       c.pos > 0 && d.a1 + warp < d.a2);
        if (op == MKBH_OP_ATTENTION) attend_ahead<T, F>(p, c.pos, d, act);
        if (d.has_vec) {
            ok = bar_wait(p, c, c.bar(kVecFull), vecs & 1u, 1);
            if (!ok) c.ctl[0] = 1;
            ++vecs;
        }
        const bool conv = (F & kRotary) && op == MKBH_OP_NORM_PROJ && L.conv_taps > 0;
        float* conv_part = conv ? L.conv_part + (size_t)g.slot * L.in_rows + d.a0 + tid : nullptr;
        const float earlier = conv && c.pos > 0 && tid < d.a1 - d.a0 ? *conv_part : 0.f;  // earlier inputs' terms
        // ---- the producers ----
        if (tid == 0 && d.wait_idx >= 0)
            poll_counter(counters + d.wait_idx, d.wait_thr, c.ctl, g.status, p.timeout_ns, i, op);
        if (!agree(c)) return;
        rec(1);
        bool signal = true;
        float kept = 0.f;  // this thread's row before the convolution
        if ((F & kClassic) && op == MKBH_OP_DELTA_STEP) {
            delta_step<T>(p, c, d, act, vec, rowv, state);
            csync();
            if (tid == 0) mbar_arrive(c.bar(kVecEmpty));
        } else if (op == MKBH_OP_ATTENTION) {
            bool done = false;
            if constexpr (sizeof(T) == 2 && (F & kRotary)) {
                done = mma_attention<T>(L);
                if (done && !attend_mma<T, F>(p, c, d, act, slot, phase)) return;
            }
            if (!done) attend_fma<T, F>(p, c.pos, d, act);
            csync();
            if (F == kClassic || L.mixer != MKBH_LATENT_ATTENTION) {  // (a latent's partial rows are merged by what expands them)
                if (tid == 0) {
                    int old;
                    int* cnt = counters + (g.num_layers + 1) * MKBH_BARRIERS_PER_LAYER + d.layer * g.max_kv_heads + d.a0;
                    asm volatile("atom.acq_rel.gpu.global.add.s32 %0, [%1], 1;" : "=r"(old) : "l"(cnt) : "memory");
                    c.ctl[1] = old == d.a2 - 1;
                }
                csync();
                signal = c.ctl[1] != 0;
                if (signal) {
                    if (F == kClassic || ((F & kClassic) && L.mixer == MKBH_DIFF_ATTENTION)) merge_splits<true>(p, c.pos, d, act);
                    else merge_splits<false>(p, c.pos, d, act);
                }
                csync();
            }
        } else if (op >= MKBH_OP_NORM_PROJ && op <= MKBH_OP_EXPAND) {
            const int rows = d.a1 - d.a0, K = d.row_bytes / (int)sizeof(T);
            // channels whose input this instruction keeps for the convolution of later tokens
            const bool canon = (F & kRotary) && op == MKBH_OP_NORM_PROJ && L.canon_taps > 1;
            const int stash_lo = canon ? (int)((long long)g.width * d.a0 / L.in_rows) : 0;
            const int stash_hi = canon ? (int)((long long)g.width * d.a1 / L.in_rows) : 0;
            const bool beside = (F & kRotary) && L.parallel, aside = op == MKBH_OP_DOWN && beside;  // the output projection adds it
            const bool adds = op == MKBH_OP_OUT_PROJ || (op == MKBH_OP_DOWN && !beside);
            float* x = (F & kRotary) ? g.x + (size_t)L.x_buf * g.width : g.x;
            const bool first = d.layer == 0 && (F == kClassic || op == MKBH_OP_ENTER || L.enter_w == nullptr);  // the stream is the embedding
            // this instruction is the only writer of its rows of the residual stream
            float old = adds && tid < rows ? ld_cg_f32(x + d.a0 + tid) : 0.f;
            if (op == MKBH_OP_OUT_PROJ && beside && L.ff && tid < rows) old += ld_cg_f32(side_out(g) + d.a0 + tid);
            if (op == MKBH_OP_OUT_PROJ) {
                if ((F & kClassic) && L.mixer == MKBH_DELTA_RULE) delta_activation(p, L, reinterpret_cast<const float*>(vec), act);
                else if (K <= 8192) plain_activation<16>(g.mixed, L.heads * L.vdim, act);
                else plain_activation<32>(g.mixed, L.heads * L.vdim, act);
            } else if ((F & kRotary) && op == MKBH_OP_DOWN && (F == kRotary || L.ff_kind == MKBH_CLAMPED_GLU)) {
                if (K <= 8192) plain_activation<16>(side_in(g), L.ff, act);
                else plain_activation<32>(side_in(g), L.ff, act);
            } else if ((F & kClassic) && op == MKBH_OP_DOWN) {
                if (K <= 8192) poly_activation<16>(p, L, act, red, turn);
                else poly_activation<32>(p, L, act, red, turn);
            } else if ((F & kRotary) && op == MKBH_OP_ABSORB) {
                plain_activation<4>(g.proj + (size_t)(d.a0 / L.rank) * (L.dim + L.rot_dim), L.dim, act);
            } else if ((F & kRotary) && op == MKBH_OP_EXPAND) {
                latent_activation(p, L, d.a0 / L.vdim, d.a2, act);
            } else if ((F & kRotary) && op == MKBH_OP_ENTER) {
                enter_activation<T>(g, first ? nullptr : g.x + (size_t)(L.x_buf ^ 1) * g.width, act);
            } else {
                const float* w = reinterpret_cast<const float*>(vec);
                const float* part = (F & kRotary) && d.part_off >= 0 ? reinterpret_cast<const float*>(c.gb + sm.vec + d.part_off) : nullptr;
                const bool in = op == MKBH_OP_NORM_PROJ;
                const float* src = first && (in || (op == MKBH_OP_NORM_UP && beside)) ? nullptr
                                   : (F & kRotary) && op == MKBH_OP_HEAD ? g.x + (size_t)p.last_buf * g.width : x;
                float* publish = src == nullptr && in && d.a0 == 0 ? x : nullptr;
                if (K <= 2048) norm_activation<T, F, 4>(p, c, src, w, part, act, red, turn, publish, stash, stash_lo, stash_hi);
                else if (K <= 8192) norm_activation<T, F, 16>(p, c, src, w, part, act, red, turn, publish, stash, stash_lo, stash_hi);
                else norm_activation<T, F, 32>(p, c, src, w, part, act, red, turn, publish, stash, stash_lo, stash_hi);
            }
            csync();
            if (tid == 0 && d.has_vec) mbar_arrive(c.bar(kVecEmpty));
            rec(2);
            const int chunks = d.row_bytes / 16;
            if (chunks <= d.groups * 32) ok = matvec_rows<T, 1>(p, c, d, act, slot, phase);
            else if (chunks <= d.groups * 64) ok = matvec_rows<T, 2>(p, c, d, act, slot, phase);
            else ok = matvec_rows<T, 4>(p, c, d, act, slot, phase);
            if (!ok) return;
            rec(3);
            unsigned long long best = 0;
            if (tid < rows) {
                float y = 0.f;
                for (int k = 0; k < d.groups; ++k) y += act[tid * d.groups + k];
                const int row = d.a0 + tid;
                kept = y;
                if (adds) {
                    x[row] = fmaf(d.row_off >= 0 ? rowv[tid] : 1.f, y, old);
                } else if (conv) {
                    g.proj[row] = fmaf(rowv[tid], y, earlier);
                } else if ((F & kRotary) && op == MKBH_OP_ENTER) {
                    x[row] = y;
                } else if (aside) {
                    side_out(g)[row] = y;
                } else if ((F & kRotary) && op == MKBH_OP_ABSORB) {
                    side_query(g)[row] = y;
                } else if ((F & kRotary) && op == MKBH_OP_EXPAND) {
                    g.mixed[row] = y;
                } else if ((F & kRotary) && op == MKBH_OP_NORM_UP && (F == kRotary || L.ff_kind == MKBH_CLAMPED_GLU)) {  // rows alternate gate, up
                    if ((tid & 1) == 0) {
                        float up = 0.f;
                        for (int k = 0; k < d.groups; ++k) up += act[(tid + 1) * d.groups + k];
                        side_in(g)[row >> 1] = clamped_glu(y, up, L.glu_limit, L.glu_alpha);
                    }
                } else if (op == MKBH_OP_HEAD) {
                    g.logits[row] = y;
                    best = argmax_key(y, row);
                } else {
                    // (NORM_UP: the stacked projection is no longer needed, its buffer takes the
                    // feed-forward's input)
                    g.proj[row] = y + (d.row_off >= 0 ? rowv[tid] : 0.f);
                }
            }
            if (op == MKBH_OP_HEAD && g.argmax_out != nullptr) {
                signal = false;
#pragma unroll
                for (int o = 16; o; o >>= 1) {
                    const unsigned long long k = __shfl_xor_sync(0xffffffffu, best, o);
                    best = k > best ? k : best;
                }
                unsigned long long* total = reinterpret_cast<unsigned long long*>(g.counters);
                if ((tid & 31) == 0 && best) atomicMax(total, best);
                csync();
                if (tid == 0) {
                    int before;
                    asm volatile("atom.acq_rel.gpu.global.add.s32 %0, [%1], 1;"
                                 : "=r"(before)
                                 : "l"(counters + d.arrive_idx)
                                 : "memory");
                    if (before == d.arrive_thr - 1)
                        *g.argmax_out = (int)(0xffffffffu - (uint32_t)(atomicMax(total, 0ull) & 0xffffffffull));
                }
            }
            csync();
        } else {
            if (tid == 0) report(g.status, c.ctl, MKBH_ERR_BAD_OPCODE, 1, i, op, 0, 0, 0);
            return;
        }
        if (tid == 0 && signal) post_signal(p, c, counters, d.arrive_idx);
        if ((F & kRotary) && op == MKBH_OP_NORM_PROJ && (L.canon_taps > 1 || L.conv_taps > 1)) {  // for later tokens only
            publish_convolutions(p, c, d, stash, kept);
            csync();
        }
        if (tid == 0) mbar_arrive(c.bar(kDescEmpty + (i & 1)));
        rec(4);
    }
}

template <typename T, int F>
__global__ void __launch_bounds__(kBlock, 1) hybrid_decode_kernel(const __grid_constant__ Params p) {
    extern __shared__ uint8_t raw[];
    const uint32_t raw32 = smem_u32(raw), base = (raw32 + 127u) & ~127u;
    const Smem sm(p.stages, p.act_bytes, p.vec_bytes);
    Cta c;
    c.base = base;
    c.gb = raw + (base - raw32);
    c.bars = base + sm.bars;
    c.ctl = reinterpret_cast<volatile int*>(c.gb + sm.ctl);
    c.instr = -1;
    c.opcode = -1;
    c.turn = 0;
    c.signals = 0;
    c.pos = p.g.pos_device ? __ldg(p.g.pos_device) : p.g.pos0;
    if (threadIdx.x == 0) {
        for (int s = 0; s < p.stages; ++s) {
            mbar_init(c.full(s), 1);
            mbar_init(c.empty(s), kConsumerWarps);
        }
        for (int s = 0; s < kRing; ++s) mbar_init(c.bar(s), 1);
        c.ctl[0] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    __syncthreads();
    if (c.pos < 0 || c.pos >= p.g.max_positions) {  // uniform over the grid
        if (threadIdx.x == 0) report(p.g.status, c.ctl, MKBH_ERR_INVALID_ARGUMENT, 1, -1, -1, c.pos, p.g.max_positions, 0);
        return;
    }
    const int warp = threadIdx.x >> 5;
    if (warp < kConsumerWarps) {
        consumer_main<T, F>(p, c, sm);
        if (kSignalWarp && threadIdx.x == 0) post_signal(p, c, nullptr, -1);
    } else if (kSignalWarp && warp == kOperandWarp + 1) {
        if ((threadIdx.x & 31) == 0) signal_main(p, c);
    }
    else if (warp == kOperandWarp) operand_main<T>(p, c, sm);
    else if constexpr (F & kRotary) loader_main<T, F>(p, c, sm);
    else if ((threadIdx.x & 31) == 0) weight_loader<T>(p, c);
    __syncthreads();
}

template <typename T, int F>
cudaError_t launch(const MkbhGlobals& g, cudaStream_t s) {
    Params p;
    p.g = g;
    p.timeout_ns = (g.wait_timeout_ms ? g.wait_timeout_ms : 2000u) * 1000000ull;
    if (!(g.flags & MKBH_FLAG_RECORD_TIMINGS)) p.g.timings = nullptr;
    int act = max(kScratchMin, 4 * pad8(g.width)), vec = 4 * g.width;
    bool part = false;
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        const bool delta = L.mixer == MKBH_DELTA_RULE;
        act = max(act, 4 * pad8(mixer_out(L)));
        if (delta) {
            act = max(act, 4 * (L.rank + 4 + L.dim));
            vec = max(vec, max(4 * L.heads * L.dim, L.dim * L.rank * (int)sizeof(T)));
        }
        if (L.ff) act = max(act, 4 * pad8(L.ff));
        if (L.enter_w) act = max(act, 4 * pad8(2 * g.width));
        part |= L.canon_taps > 1;
    }
    // keys staged at a time: 64, fewer when a tile of wide heads would not fit
    p.attn_chunk = 64;
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        if (!is_attention(L)) continue;
        const int per = L.heads / L.kv_heads, nq = attn_maps(L) * per;
        act = max(act, max(4 * merge_scratch_floats(nq, g.max_splits, per, attn_vdim(L)),
                           mma_attention<T>(L) ? 4 * MmaScratch(L).total : attn_scratch_bytes<T>(L, 8)));
    }
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        if (!is_attention(L) || mma_attention<T>(L)) continue;
        while (p.attn_chunk > 8 && attn_scratch_bytes<T>(L, p.attn_chunk) > act) p.attn_chunk -= 8;
    }
    p.last_buf = g.layers_host[g.num_layers - 1].x_buf;
    p.act_bytes = (act + 127) & ~127;
    p.part_base = (vec + 32 + 127) & ~127;
    p.vec_bytes = p.part_base + (part ? (4 * g.width + 32 + 127) & ~127 : 0);
    const int fixed = Smem(0, p.act_bytes, p.vec_bytes).total + 128;
    p.stages = (kSmemLimit - fixed) / kStage;
    if (p.stages > kMaxStages) p.stages = kMaxStages;
    if (p.stages < 2) return cudaErrorInvalidValue;
    const int smem = Smem(p.stages, p.act_bytes, p.vec_bytes).total + 128;
    static int set[64] = {};
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    if (set[dev & 63] < smem) {
        e = cudaFuncSetAttribute(hybrid_decode_kernel<T, F>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return e;
        set[dev & 63] = smem;
    }
    e = cudaMemsetAsync(g.counters, 0, (size_t)g.num_counters * 4, s);
    if (e != cudaSuccess) return e;
    // cooperative: the CTAs wait for one another, so all of them must be resident
    void* args[] = {&p};
    return cudaLaunchCooperativeKernel((const void*)hybrid_decode_kernel<T, F>, dim3(g.num_sms), dim3(kBlock), args,
                                       (size_t)smem, s);
}

}  // namespace

template <>
cudaError_t decode_build<MKBH_FEATURES>(const MkbhGlobals& g, cudaStream_t s) {
    return g.dtype == MKBH_F32 ? launch<float, MKBH_FEATURES>(g, s) : launch<bf16, MKBH_FEATURES>(g, s);
}

#if MKBH_FEATURES == 1
cudaError_t decode_launch(const MkbhGlobals& g, cudaStream_t s) {
    int features = g.norm_kind == MKBH_LAYER_NORM ? kClassic : kRotary;
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        features |= L.mixer == MKBH_DELTA_RULE || L.mixer == MKBH_DIFF_ATTENTION ? kClassic : kRotary;
        if (L.ff) features |= L.ff_kind == MKBH_POLY_NORM ? kClassic : kRotary;
        if (L.parallel || L.canon_taps || L.conv_taps || L.enter_w) features |= kRotary;
    }
    return features == kClassic ? decode_build<kClassic>(g, s) : features == kRotary ? decode_build<kRotary>(g, s) : decode_build<kClassic | kRotary>(g, s);
}
#endif

}  // namespace mkbh
