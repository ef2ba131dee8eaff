// C ABI of libmkb200_hybrid.so (include/mkb200_hybrid.h): host-side validation, the prefill
// sequence, launches and status read-back.
#include <cstdarg>
#include <cstdio>
#include <cstring>

#include "hybrid_kernels.h"

namespace {

using namespace mkbh;

thread_local char g_error[512] = "";

int fail(int code, const char* fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_error, sizeof(g_error), fmt, ap);
    va_end(ap);
    return code;
}

#define MKBH_TRY(call)                                                                             \
    do {                                                                                           \
        cudaError_t e_ = (call);                                                                   \
        if (e_ != cudaSuccess) return fail(MKBH_ERR_CUDA, "%s: %s", #call, cudaGetErrorString(e_)); \
    } while (0)

#define REQUIRE(cond, ...)                                            \
    do {                                                              \
        if (!(cond)) return fail(MKBH_ERR_INVALID_ARGUMENT, __VA_ARGS__); \
    } while (0)

int elem_bytes(const MkbhGlobals& g) { return g.dtype == MKBH_F32 ? 4 : 2; }

int out_features(const MkbhLayer& L) { return L.heads * (L.mixer == MKBH_DELTA_RULE ? L.dim : L.vdim); }

int check_layer(const MkbhGlobals& g, int i) {
    const MkbhLayer& L = g.layers_host[i];
    const bool delta = L.mixer == MKBH_DELTA_RULE;
    REQUIRE(delta || L.mixer == MKBH_DIFF_ATTENTION, "layer %d: unknown mixer %d", i, L.mixer);
    REQUIRE(L.heads > 0 && L.dim > 0, "layer %d: heads and dim must be positive", i);
    REQUIRE(L.in_w && L.out_w && L.norm1 && L.ls1, "layer %d: missing weights", i);
    if (delta) {
        REQUIRE(L.dim <= 256, "layer %d: recurrence head size %d > 256", i, L.dim);
        REQUIRE(L.rank > 0 && L.rank <= 256, "layer %d: decay rank %d outside 1..256", i, L.rank);
        REQUIRE(L.decay_w2 && L.decay_w0 && L.out_norm && L.state, "layer %d: incomplete recurrence", i);
        REQUIRE(L.in_rows == 5 * L.heads * L.dim + L.rank, "layer %d: %d projection rows", i, L.in_rows);
    } else {
        REQUIRE(L.kv_heads > 0 && L.heads % L.kv_heads == 0, "layer %d: %d heads over %d KV heads", i, L.heads, L.kv_heads);
        REQUIRE(L.vdim > 0 && L.vdim <= 512, "layer %d: value size %d outside 1..512", i, L.vdim);
        REQUIRE(L.window > 0 && L.keep_first >= 0, "layer %d: window %d, kept %d", i, L.window, L.keep_first);
        REQUIRE(L.cache_keep >= L.keep_first && L.cache_ring > 0, "layer %d: cache too small", i);
        REQUIRE(L.cache_keep + L.cache_ring >= g.max_positions || L.cache_ring >= L.window + g.portion_capacity,
                "layer %d: a ring of %d rows cannot hold the window and a portion", i, L.cache_ring);
        REQUIRE(L.k_cache && L.v_cache, "layer %d: no cache", i);
        REQUIRE(2 * (L.heads / L.kv_heads) <= 16 * (512 / L.vdim), "layer %d: too many query heads per KV head", i);
        REQUIRE(L.in_rows == L.heads * (2 * L.dim + L.vdim) + (L.owns_kv ? L.kv_heads * (2 * L.dim + L.vdim) : 0),
                "layer %d: %d projection rows", i, L.in_rows);
    }
    if (L.ff) REQUIRE(L.ff > 0 && L.up_w && L.down_w && L.norm2 && L.ls2, "layer %d: incomplete feed-forward", i);
    const int widest = pad8(L.ff > out_features(L) ? L.ff : out_features(L));
    REQUIRE((widest > pad8(g.width) ? widest : pad8(g.width)) * elem_bytes(g) <= kMaxRowBytes,
            "layer %d: a weight row is longer than %d bytes", i, kMaxRowBytes);
    return MKBH_OK;
}

int check_globals(const MkbhGlobals* gp) {
    REQUIRE(gp != nullptr, "null globals");
    const MkbhGlobals& g = *gp;
    REQUIRE(g.abi_version == MKBH_ABI_VERSION && g.struct_bytes == sizeof(MkbhGlobals), "ABI mismatch (version %u, %u bytes; expected %d, %zu)",
            g.abi_version, g.struct_bytes, MKBH_ABI_VERSION, sizeof(MkbhGlobals));
    REQUIRE(g.dtype == MKBH_BF16 || g.dtype == MKBH_F32, "unknown dtype %d", g.dtype);
    REQUIRE(g.num_layers > 0 && g.width > 0 && g.vocab > 0 && g.max_positions > 0 && g.slots > 0, "empty model");
    REQUIRE(g.slot >= 0 && g.slot < g.slots, "slot %d of %d", g.slot, g.slots);
    REQUIRE(g.embed && g.pos && g.head && g.final_norm && g.layers_host && g.layers_device && g.tokens && g.status,
            "missing pointers");
    REQUIRE(g.x && g.proj && g.mixed && g.decay && g.act, "missing activation buffers");
    for (int i = 0; i < g.num_layers; ++i)
        if (int rc = check_layer(g, i)) return rc;
    return MKBH_OK;
}

template <typename T>
cudaError_t gemm(const MkbhGlobals& g, int64_t lda, const void* W, int T_, int N, int K, const GemmEpilogue& e, cudaStream_t s) {
    const int Kp = pad8(K);
    if constexpr (sizeof(T) == 4) return gemm_f32(static_cast<const float*>(g.act), lda, static_cast<const float*>(W), Kp, T_, N, Kp, e, s);
    else return gemm_bf16(static_cast<const bf16*>(g.act), lda, static_cast<const bf16*>(W), Kp, T_, N, Kp, e, g.status, s);
}

template <typename T>
int prefill(const MkbhGlobals& g, cudaStream_t s) {
    using P = Prefill<T>;
    T* act = static_cast<T*>(g.act);
    const int n = g.num_tokens, width = g.width;
    MKBH_TRY(P::embed(g, s));
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        const int64_t ldx = pad8(width), ldp = pad8(L.in_rows);
        MKBH_TRY(P::norm(g.x, nullptr, n, width, L.norm1, g.eps, act, ldx, s));
        MKBH_TRY(gemm<T>(g, ldx, L.in_w, n, L.in_rows, width, GemmEpilogue{g.proj, ldp, L.in_bias, nullptr}, s));
        const int K = out_features(L);
        if (L.mixer == MKBH_DELTA_RULE) MKBH_TRY(P::delta(g, L, act, pad8(K), s));
        else MKBH_TRY(P::attention(g, L, act, pad8(K), s));
        MKBH_TRY(gemm<T>(g, pad8(K), L.out_w, n, width, K, GemmEpilogue{g.x, width, nullptr, L.ls1}, s));
        if (L.ff) {
            MKBH_TRY(P::norm(g.x, nullptr, n, width, L.norm2, g.eps, act, ldx, s));
            MKBH_TRY(gemm<T>(g, ldx, L.up_w, n, L.ff, width, GemmEpilogue{g.proj, pad8(L.ff), nullptr, nullptr}, s));
            MKBH_TRY(P::poly_norm(g.proj, pad8(L.ff), n, L.ff, L.act, g.eps, act, pad8(L.ff), s));
            MKBH_TRY(gemm<T>(g, pad8(L.ff), L.down_w, n, width, L.ff, GemmEpilogue{g.x, width, nullptr, L.ls2}, s));
        }
        if (g.layers_out)
            MKBH_TRY(cudaMemcpyAsync(g.layers_out + (size_t)i * n * width, g.x, (size_t)n * width * 4, cudaMemcpyDeviceToDevice, s));
    }
    if (g.num_want > 0) {
        MKBH_TRY(P::norm(g.x, g.want_rows, g.num_want, width, g.final_norm, g.eps, act, pad8(width), s));
        MKBH_TRY(gemm<T>(g, pad8(width), g.head, g.num_want, g.vocab, width, GemmEpilogue{g.logits, g.vocab, nullptr, nullptr}, s));
    }
    return MKBH_OK;
}

}  // namespace

extern "C" {

int mkb_hybrid_prefill(const MkbhGlobals* gp, void* stream) {
    if (int rc = check_globals(gp)) return rc;
    const MkbhGlobals& g = *gp;
    const int n = g.num_tokens;
    REQUIRE(n > 0 && n <= g.portion_capacity, "a portion of %d tokens (capacity %d)", n, g.portion_capacity);
    REQUIRE(g.pos0 >= 0 && g.pos0 + n <= g.max_positions, "positions %d..%d of %d", g.pos0, g.pos0 + n - 1, g.max_positions);
    REQUIRE(g.num_want >= 0 && g.num_want <= n && (g.num_want == 0 || (g.want_rows && g.logits)), "bad list of wanted rows");
    int64_t proj = 0, mixed = 0, decay = 0, act = pad8(g.width);
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        const int64_t out = pad8(out_features(L));
        if (pad8(L.in_rows) > proj) proj = pad8(L.in_rows);
        if (pad8(L.ff) > proj) proj = pad8(L.ff);
        if (out > mixed) mixed = out;
        if (L.mixer == MKBH_DELTA_RULE && L.heads * (L.dim + 2) > decay) decay = L.heads * (L.dim + 2);
        if (out > act) act = out;
        if (pad8(L.ff) > act) act = pad8(L.ff);
    }
    REQUIRE(g.x_elems >= (int64_t)n * g.width && g.proj_elems >= n * proj && g.mixed_elems >= n * mixed && g.act_elems >= n * act &&
                g.decay_elems >= n * decay,
            "activation buffers are too small for %d tokens", n);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    return g.dtype == MKBH_F32 ? prefill<float>(g, s) : prefill<bf16>(g, s);
}

int mkb_hybrid_decode(const MkbhGlobals* gp, void* stream) {
    if (int rc = check_globals(gp)) return rc;
    const MkbhGlobals& g = *gp;
    REQUIRE(g.pos_device || (g.pos0 >= 0 && g.pos0 < g.max_positions), "position %d of %d", g.pos0, g.max_positions);
    REQUIRE(g.instructions && g.arrivals && g.counters && g.logits && g.queue_len > 0, "missing schedule");
    REQUIRE(g.num_counters >= 2 + (g.num_layers + 1) * MKBH_BARRIERS_PER_LAYER + g.num_layers * g.max_kv_heads, "too few counters");
    REQUIRE(((uintptr_t)g.counters & 7) == 0, "counters must be 8-byte aligned");
    int sms = 0, dev = 0;
    MKBH_TRY(cudaGetDevice(&dev));
    MKBH_TRY(cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev));
    REQUIRE(g.num_sms > 0 && g.num_sms <= sms, "%d instruction queues on %d SMs", g.num_sms, sms);
    for (int i = 0; i < g.num_layers; ++i)
        if (g.layers_host[i].mixer == MKBH_DIFF_ATTENTION)
            REQUIRE(g.attn_part && g.max_splits >= 1 && g.max_splits <= 32 && g.part_vdim >= g.layers_host[i].vdim &&
                        g.layers_host[i].kv_heads <= g.max_kv_heads,
                    "attention scratch too small");
    MKBH_TRY(decode_launch(g, static_cast<cudaStream_t>(stream)));
    return MKBH_OK;
}

int mkb_hybrid_validate(const MkbhGlobals* gp, const int32_t* ins) {
    if (int rc = check_globals(gp)) return rc;
    const MkbhGlobals& g = *gp;
    REQUIRE(ins && g.num_sms > 0 && g.queue_len > 0, "no instructions");
    for (int q = 0; q < g.num_sms; ++q)
        for (int k = 0; k < g.queue_len; ++k) {
            const int32_t* w = ins + ((size_t)q * g.queue_len + k) * MKBH_INTS_PER_INSTRUCTION;
            const int op = w[0], layer = w[1];
            if (op == MKBH_OP_NOOP) continue;
            REQUIRE(op >= 1 && op <= MKBH_OP_HEAD, "queue %d, instruction %d: opcode %d", q, k, op);
            REQUIRE(layer >= 0 && layer < g.num_layers, "queue %d, instruction %d: layer %d", q, k, layer);
            const MkbhLayer& L = g.layers_host[layer];
            if (op == MKBH_OP_DELTA_STEP) {
                REQUIRE(L.mixer == MKBH_DELTA_RULE && w[2] >= 0 && w[2] < L.heads && w[3] >= 0 && w[3] < w[4] && w[4] <= L.dim,
                        "queue %d, instruction %d: head %d, columns %d..%d", q, k, w[2], w[3], w[4]);
            } else if (op == MKBH_OP_ATTENTION) {
                REQUIRE(L.mixer == MKBH_DIFF_ATTENTION && w[2] >= 0 && w[2] < L.kv_heads && w[3] >= 0 && w[3] < w[4] && w[4] <= g.max_splits,
                        "queue %d, instruction %d: KV head %d, split %d of %d", q, k, w[2], w[3], w[4]);
            } else {
                int rows, K;
                if (op == MKBH_OP_NORM_PROJ) rows = L.in_rows, K = g.width;
                else if (op == MKBH_OP_OUT_PROJ) rows = g.width, K = out_features(L);
                else if (op == MKBH_OP_HEAD) rows = g.vocab, K = g.width;
                else {
                    REQUIRE(L.ff > 0, "queue %d, instruction %d: layer %d has no feed-forward", q, k, layer);
                    rows = op == MKBH_OP_NORM_UP ? L.ff : g.width;
                    K = op == MKBH_OP_NORM_UP ? g.width : L.ff;
                }
                const int chunks = pad8(K) * elem_bytes(g) / 16;
                int groups = 1;
                while (groups < 16 && groups * 32 < chunks) groups *= 2;
                REQUIRE(w[2] >= 0 && w[2] < w[3] && w[3] <= rows && w[3] - w[2] <= 512 && (w[3] - w[2]) * groups <= 4096,
                        "queue %d, instruction %d: rows %d..%d of %d", q, k, w[2], w[3], rows);
            }
        }
    return MKBH_OK;
}

int mkb_hybrid_sync_status(const MkbhGlobals* gp, void* stream, int32_t out[MKBH_STATUS_WORDS]) {
    REQUIRE(gp && gp->status && out, "null argument");
    MKBH_TRY(cudaStreamSynchronize(static_cast<cudaStream_t>(stream)));
    MKBH_TRY(cudaMemcpy(out, gp->status, MKBH_STATUS_WORDS * 4, cudaMemcpyDeviceToHost));
    if (out[0] != MKBH_OK) MKBH_TRY(cudaMemset(gp->status, 0, MKBH_STATUS_WORDS * 4));
    return out[0];
}

const char* mkb_hybrid_last_error(void) { return g_error; }
int mkb_hybrid_abi_version(void) { return MKBH_ABI_VERSION; }
size_t mkb_hybrid_layer_bytes(void) { return sizeof(MkbhLayer); }
size_t mkb_hybrid_globals_bytes(void) { return sizeof(MkbhGlobals); }

}  // extern "C"
