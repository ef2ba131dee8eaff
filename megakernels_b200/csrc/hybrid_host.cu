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

int check_attention(const MkbhGlobals& g, const MkbhLayer& L, int i) {
    const bool diff = L.mixer == MKBH_DIFF_ATTENTION, latent = L.mixer == MKBH_LATENT_ATTENTION;
    REQUIRE(L.kv_heads > 0 && L.heads % L.kv_heads == 0, "layer %d: %d heads over %d KV heads", i, L.heads, L.kv_heads);
    REQUIRE(L.vdim > 0 && L.vdim <= 512, "layer %d: value size %d outside 1..512", i, L.vdim);
    REQUIRE(L.window > 0 && L.keep_first >= 0 && L.chunk >= 0, "layer %d: window %d, kept %d, chunk %d", i, L.window, L.keep_first, L.chunk);
    REQUIRE(L.cache_keep >= L.keep_first && L.cache_ring > 0, "layer %d: cache too small", i);
    REQUIRE((int64_t)L.cache_keep + L.cache_ring >= g.max_positions || L.cache_ring >= (int64_t)L.window + g.portion_capacity,
            "layer %d: a ring of %d rows cannot hold the window and a portion", i, L.cache_ring);
    REQUIRE(L.k_cache && (latent || L.v_cache), "layer %d: no cache", i);
    const int evs = latent ? L.rank : L.vdim;
    REQUIRE(evs > 0 && evs <= 512, "layer %d: value size %d outside 1..512", i, evs);
    REQUIRE((diff ? 2 : 1) * (L.heads / L.kv_heads) <= 16 * (512 / evs), "layer %d: too many query heads per KV head", i);
    if (diff) {
        REQUIRE(L.chunk == 0 && L.in_rows == L.heads * (2 * L.dim + L.vdim) + (L.owns_kv ? L.kv_heads * (2 * L.dim + L.vdim) : 0),
                "layer %d: %d projection rows", i, L.in_rows);
        return MKBH_OK;
    }
    REQUIRE(L.dim <= 512, "layer %d: head size %d > 512", i, L.dim);
    REQUIRE(L.rope && L.rope_dims >= 0 && L.rope_dims % 2 == 0 && L.rope_dims <= (latent ? L.rot_dim : L.dim),
            "layer %d: %d rotated dimensions", i, L.rope_dims);
    REQUIRE(g.query && g.side, "layer %d: missing buffers", i);
    if (latent) {
        REQUIRE(L.rot_dim > 0 && L.rot_dim <= 512 && L.k_norm && L.absorb_w && L.expand_w && g.keys, "layer %d: incomplete latent attention", i);
        REQUIRE(L.cache_keep == 0 && L.cache_ring >= g.max_positions && L.window >= g.max_positions && L.chunk == 0 && L.conv_taps == 0,
                "layer %d: latent attention is causal over all positions", i);
        REQUIRE(L.in_rows == L.heads * (L.dim + L.rot_dim) + L.rank + L.rot_dim, "layer %d: %d projection rows", i, L.in_rows);
        REQUIRE(g.side_rank >= L.heads * L.rank, "layer %d: missing buffers", i);
    } else {
        REQUIRE(L.q_norm && L.k_norm && L.temp, "layer %d: incomplete attention", i);
        REQUIRE(!L.value_rope || L.vdim % 2 == 0, "layer %d: rotated values of odd size %d", i, L.vdim);
        REQUIRE(L.in_rows == L.heads * L.dim + L.kv_heads * (L.dim + L.vdim), "layer %d: %d projection rows", i, L.in_rows);
    }
    return MKBH_OK;
}

int check_layer(const MkbhGlobals& g, int i) {
    const MkbhLayer& L = g.layers_host[i];
    const bool delta = L.mixer == MKBH_DELTA_RULE;
    REQUIRE(L.mixer >= MKBH_DELTA_RULE && L.mixer <= MKBH_LATENT_ATTENTION, "layer %d: unknown mixer %d", i, L.mixer);
    REQUIRE(L.heads > 0 && L.dim > 0, "layer %d: heads and dim must be positive", i);
    REQUIRE(L.in_w && L.out_w && L.norm1, "layer %d: missing weights", i);
    if (delta) {
        REQUIRE(L.dim <= 256, "layer %d: recurrence head size %d > 256", i, L.dim);
        REQUIRE(L.rank > 0 && L.rank <= 256, "layer %d: decay rank %d outside 1..256", i, L.rank);
        REQUIRE(L.decay_w2 && L.decay_w0 && L.out_norm && L.state, "layer %d: incomplete recurrence", i);
        REQUIRE(L.in_rows == 5 * L.heads * L.dim + L.rank, "layer %d: %d projection rows", i, L.in_rows);
    } else if (int rc = check_attention(g, L, i)) {
        return rc;
    }
    if (L.ff) {
        REQUIRE(L.ff > 0 && L.up_w && L.down_w && L.norm2, "layer %d: incomplete feed-forward", i);
        REQUIRE(L.ff_kind == MKBH_POLY_NORM || L.ff_kind == MKBH_CLAMPED_GLU, "layer %d: unknown feed-forward %d", i, L.ff_kind);
        REQUIRE(L.ff_kind == MKBH_CLAMPED_GLU || !L.parallel, "layer %d: this feed-forward does not run beside a mixer", i);
        if (L.ff_kind == MKBH_CLAMPED_GLU)
            REQUIRE(g.act2 && g.ffn && g.side && g.side_ff >= L.ff, "layer %d: missing feed-forward buffers", i);
    }
    REQUIRE(L.x_buf == 0 || L.x_buf == 1, "layer %d: residual buffer %d", i, L.x_buf);
    if (i > 0) REQUIRE(L.x_buf == (g.layers_host[i - 1].x_buf ^ (L.enter_w ? 1 : 0)), "layer %d: residual buffer %d", i, L.x_buf);
    REQUIRE(L.canon_taps >= 0 && L.conv_taps >= 0 && (L.conv_taps == 0 || L.mixer == MKBH_ATTENTION), "layer %d: convolutions", i);
    if (L.canon_taps)
        REQUIRE(L.canon_w && L.canon_gain && L.canon_hist && L.canon_part && g.tail && L.canon_taps * g.width * 4 <= 200 * 1024,
                "layer %d: incomplete or oversized input convolution", i);
    if (L.conv_taps) REQUIRE(L.conv_w && L.conv_hist && L.conv_part && !L.in_bias, "layer %d: incomplete convolution", i);
    int widest = L.ff > mixer_out(L) ? L.ff : mixer_out(L);
    if (L.enter_w && 2 * g.width > widest) widest = 2 * g.width;
    if (g.width > widest) widest = g.width;
    REQUIRE(pad8(widest) * elem_bytes(g) <= kMaxRowBytes, "layer %d: a weight row is longer than %d bytes", i, kMaxRowBytes);
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
    REQUIRE(g.embed && g.head && g.final_norm && g.layers_host && g.layers_device && g.tokens && g.status,
            "missing pointers");
    REQUIRE(g.x && g.proj && g.mixed && g.decay && g.act, "missing activation buffers");
    REQUIRE(g.norm_kind == MKBH_LAYER_NORM || g.norm_kind == MKBH_RMS_NORM, "unknown norm %d", g.norm_kind);
    REQUIRE(g.side_ff % 8 == 0 && g.side_rank % 8 == 0 && (!g.side || g.side_elems >= (int64_t)g.side_ff + pad8(g.width) + (int64_t)g.side_rank),
            "side buffer too small");
    for (int i = 0; i < g.num_layers; ++i)
        if (int rc = check_layer(g, i)) return rc;
    return MKBH_OK;
}

template <typename T>
cudaError_t gemm(const MkbhGlobals& g, const T* A, int64_t lda, const void* W, int T_, int N, int K, const GemmEpilogue& e, cudaStream_t s) {
    if constexpr (sizeof(T) == 4) return gemm_f32(A, lda, static_cast<const float*>(W), pad8(K), T_, N, K, e, s);
    else return gemm_bf16(A, lda, static_cast<const bf16*>(W), pad8(K), T_, N, K, e, g.status, s);
}

template <typename T>
int feed_forward(const MkbhGlobals& g, const MkbhLayer& L, cudaStream_t s) {
    using P = Prefill<T>;
    const int n = g.num_tokens, width = g.width;
    const int64_t ldx = pad8(width), ldf = pad8(L.ff);
    T* act = static_cast<T*>(g.act);
    MKBH_TRY(P::norm(g, nullptr, n, L.norm2, act, ldx, s));
    T* inner = act;
    if (L.ff_kind == MKBH_CLAMPED_GLU) {
        inner = static_cast<T*>(g.ffn);
        MKBH_TRY(gemm<T>(g, act, ldx, L.up_w, n, up_rows(L), width, GemmEpilogue::glu(inner, ldf, L.glu_limit, L.glu_alpha), s));
    } else {
        MKBH_TRY(gemm<T>(g, act, ldx, L.up_w, n, L.ff, width, GemmEpilogue::store(g.proj, ldf, nullptr), s));
        MKBH_TRY(P::poly_norm(g.proj, ldf, n, L.ff, L.act, g.eps, inner, ldf, s));
    }
    MKBH_TRY(gemm<T>(g, inner, ldf, L.down_w, n, width, L.ff, GemmEpilogue::add(g.x, width, L.ls2), s));
    return MKBH_OK;
}

template <typename T>
int prefill(const MkbhGlobals& g, cudaStream_t s) {
    using P = Prefill<T>;
    T *act = static_cast<T*>(g.act), *act2 = static_cast<T*>(g.act2), *ffn = static_cast<T*>(g.ffn);
    const int n = g.num_tokens, width = g.width;
    MKBH_TRY(P::embed(g, s));
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        const int64_t ldx = pad8(width), ldp = pad8(L.in_rows), ldf = pad8(L.ff);
        const bool beside = L.ff && L.parallel;
        if (L.enter_w) {
            MKBH_TRY(P::enter(g, act, pad8(2 * width), s));
            MKBH_TRY(gemm<T>(g, act, pad8(2 * width), L.enter_w, n, width, 2 * width, GemmEpilogue::store(g.x, width, nullptr), s));
        }
        if (L.canon_taps || beside) MKBH_TRY(P::canon_norm(g, L, act, beside ? act2 : nullptr, ldx, s));
        else MKBH_TRY(P::norm(g, nullptr, n, L.norm1, act, ldx, s));
        MKBH_TRY(gemm<T>(g, act, ldx, L.in_w, n, L.in_rows, width, GemmEpilogue::store(g.proj, ldp, L.in_bias), s));
        if (beside) MKBH_TRY(gemm<T>(g, act2, ldx, L.up_w, n, up_rows(L), width, GemmEpilogue::glu(ffn, ldf, L.glu_limit, L.glu_alpha), s));
        const int K = mixer_out(L);
        if (L.mixer == MKBH_DELTA_RULE) {
            MKBH_TRY(P::delta(g, L, act, pad8(K), s));
        } else if (L.mixer == MKBH_DIFF_ATTENTION) {
            MKBH_TRY(P::attention(g, L, act, pad8(K), s));
        } else {
            MKBH_TRY(P::rotary_operands(g, L, s));
            if (L.mixer == MKBH_LATENT_ATTENTION) {  // keys and values of all heads and positions so far
                const int64_t lr = latent_row(L), ldk = pad8(L.heads * (L.dim + L.vdim));
                const T* latents = static_cast<const T*>(L.k_cache) + (size_t)g.slot * L.cache_ring * lr;
                MKBH_TRY(gemm<T>(g, latents, lr, L.expand_w, g.pos0 + n, L.heads * (L.dim + L.vdim), L.rank, GemmEpilogue::to(g.keys, ldk), s));
            }
            MKBH_TRY(P::rotary_attention(g, L, act, pad8(K), s));
        }
        if (L.canon_taps > 1 || L.conv_taps > 1) MKBH_TRY(P::keep_inputs(g, L, s));
        MKBH_TRY(gemm<T>(g, act, pad8(K), L.out_w, n, width, K, GemmEpilogue::add(g.x, width, L.ls1), s));
        if (beside) MKBH_TRY(gemm<T>(g, ffn, ldf, L.down_w, n, width, L.ff, GemmEpilogue::add(g.x, width, L.ls2), s));
        else if (L.ff)
            if (int rc = feed_forward<T>(g, L, s)) return rc;
        if (g.layers_out)
            MKBH_TRY(cudaMemcpyAsync(g.layers_out + (size_t)i * n * width, g.x, (size_t)n * width * 4, cudaMemcpyDeviceToDevice, s));
    }
    if (g.num_want > 0) {
        MKBH_TRY(P::norm(g, g.want_rows, g.num_want, g.final_norm, act, pad8(width), s));
        MKBH_TRY(gemm<T>(g, act, pad8(width), g.head, g.num_want, g.vocab, width, GemmEpilogue::store(g.logits, g.vocab, nullptr), s));
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
    int64_t proj = 0, mixed = 0, decay = 0, act = pad8(g.width), query = 0, act2 = 0, ffn = 0, keys = 0, tail = 0;
    auto most = [](int64_t& a, int64_t b) { if (b > a) a = b; };
    for (int i = 0; i < g.num_layers; ++i) {
        const MkbhLayer& L = g.layers_host[i];
        const int64_t out = pad8(mixer_out(L));
        most(proj, pad8(L.in_rows));
        if (L.ff && L.ff_kind == MKBH_POLY_NORM) most(proj, pad8(L.ff)), most(act, pad8(L.ff));
        if (L.ff && L.ff_kind == MKBH_CLAMPED_GLU) most(ffn, pad8(L.ff)), most(act2, pad8(g.width));
        most(mixed, out);
        if (L.mixer == MKBH_DELTA_RULE) most(decay, L.heads * (L.dim + 2));
        most(act, out);
        if (L.enter_w) most(act, pad8(2 * g.width));
        if (L.mixer == MKBH_ATTENTION || L.mixer == MKBH_LATENT_ATTENTION)
            most(query, pad8(L.heads * (g.dtype == MKBH_F32 ? query_head<float>(L) : query_head<bf16>(L))));
        if (L.mixer == MKBH_LATENT_ATTENTION) {
            most(keys, pad8(L.heads * (L.dim + L.vdim)));
        }
        if (L.canon_taps) most(tail, (int64_t)L.canon_taps * g.width);
    }
    REQUIRE(g.x_elems >= (int64_t)n * g.width && g.proj_elems >= n * proj && g.mixed_elems >= n * mixed && g.act_elems >= n * act &&
                g.decay_elems >= n * decay && g.query_elems >= n * query && g.act2_elems >= n * act2 && g.ffn_elems >= n * ffn &&
                g.keys_elems >= (g.pos0 + n) * keys && g.tail_elems >= tail,
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
        if (is_attention(g.layers_host[i])) {
            const MkbhLayer& L = g.layers_host[i];
            REQUIRE(g.attn_part && g.max_splits >= 1 && g.max_splits <= 64 &&
                        g.part_vdim >= (L.mixer == MKBH_LATENT_ATTENTION ? L.rank : L.vdim) && L.kv_heads <= g.max_kv_heads,
                    "attention scratch too small");
        }
    REQUIRE(g.x_elems >= 2 * (int64_t)g.width, "residual buffers too small");
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
            REQUIRE(op >= 1 && op <= MKBH_OP_EXPAND, "queue %d, instruction %d: opcode %d", q, k, op);
            REQUIRE(layer >= 0 && layer < g.num_layers, "queue %d, instruction %d: layer %d", q, k, layer);
            const MkbhLayer& L = g.layers_host[layer];
            if (op == MKBH_OP_DELTA_STEP) {
                REQUIRE(L.mixer == MKBH_DELTA_RULE && w[2] >= 0 && w[2] < L.heads && w[3] >= 0 && w[3] < w[4] && w[4] <= L.dim,
                        "queue %d, instruction %d: head %d, columns %d..%d", q, k, w[2], w[3], w[4]);
            } else if (op == MKBH_OP_ATTENTION) {
                REQUIRE(is_attention(L) && w[2] >= 0 && w[2] < L.kv_heads && w[3] >= 0 && w[3] < w[4] && w[4] <= g.max_splits &&
                            (w[4] <= 32 || L.mixer == MKBH_LATENT_ATTENTION),
                        "queue %d, instruction %d: KV head %d, split %d of %d", q, k, w[2], w[3], w[4]);
            } else {
                int rows, K;
                if (op == MKBH_OP_NORM_PROJ) rows = L.in_rows, K = g.width;
                else if (op == MKBH_OP_OUT_PROJ) rows = g.width, K = mixer_out(L);
                else if (op == MKBH_OP_HEAD) rows = g.vocab, K = g.width;
                else if (op == MKBH_OP_ENTER) {
                    REQUIRE(L.enter_w, "queue %d, instruction %d: layer %d starts no pass", q, k, layer);
                    rows = g.width, K = 2 * g.width;
                } else if (op == MKBH_OP_ABSORB || op == MKBH_OP_EXPAND) {
                    REQUIRE(L.mixer == MKBH_LATENT_ATTENTION, "queue %d, instruction %d: layer %d has no latent", q, k, layer);
                    const int per = op == MKBH_OP_ABSORB ? L.rank : L.vdim;  // rows of a head
                    rows = L.heads * per, K = op == MKBH_OP_ABSORB ? L.dim : L.rank;
                    if (op == MKBH_OP_EXPAND)
                        REQUIRE(w[4] > 0 && w[4] <= g.max_splits, "queue %d, instruction %d: %d splits", q, k, w[4]);
                    REQUIRE(w[2] >= 0 && w[2] < w[3] && w[2] / per == (w[3] - 1) / per, "queue %d, instruction %d: rows %d..%d of several heads", q, k, w[2], w[3]);
                } else {
                    REQUIRE(L.ff > 0, "queue %d, instruction %d: layer %d has no feed-forward", q, k, layer);
                    rows = op == MKBH_OP_NORM_UP ? up_rows(L) : g.width;
                    K = op == MKBH_OP_NORM_UP ? g.width : L.ff;
                    if (op == MKBH_OP_NORM_UP && L.ff_kind == MKBH_CLAMPED_GLU)
                        REQUIRE(w[2] % 2 == 0 && w[3] % 2 == 0, "queue %d, instruction %d: rows %d..%d split a gated unit", q, k, w[2], w[3]);
                }
                if (op == MKBH_OP_NORM_PROJ && L.canon_taps > 1)
                    REQUIRE((int64_t)g.width * w[3] / L.in_rows - (int64_t)g.width * w[2] / L.in_rows <= 512,
                            "queue %d, instruction %d: rows %d..%d carry too many channels", q, k, w[2], w[3]);
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
