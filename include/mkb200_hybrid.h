/*
 * C ABI of libmkb200_hybrid.so: decoders whose layers are listed one by one, each with a
 * mixer (generalized delta rule, windowed differential attention, rotary attention in chunks,
 * latent attention) and an optional feed-forward, after the mixer or beside it.  A stretch of
 * layers may run several times: the descriptors below are layer RUNS, with state of their own,
 * that may share weights.  Plain pointers and sizes; no framework type crosses it.
 *
 * Two entry points do the work, both asynchronous on the given stream:
 *   mkb_hybrid_decode   one token of one sequence, ONE persistent kernel launch that
 *                       interprets per-SM instruction queues (as mkb_launch does);
 *   mkb_hybrid_prefill  a portion of 1..portion_capacity tokens of one sequence, a sequence
 *                       of tensor-core / scan / attention kernels.
 * Both read and advance the same per-slot state (key/value rows, recurrent
 * matrices, the last inputs of short convolutions), so a
 * sequence may be cut into portions and single tokens in any way.
 */
#ifndef MKB200_HYBRID_H
#define MKB200_HYBRID_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define MKBH_ABI_VERSION 2

enum MkbhCode { /* same values as MkbCode of mkb200.h */
    MKBH_OK = 0,
    MKBH_ERR_INVALID_ARGUMENT = 1,
    MKBH_ERR_CUDA = 2,
    MKBH_ERR_DEVICE_TIMEOUT = 3,
    MKBH_ERR_BAD_OPCODE = 4,
    MKBH_ERR_UNSUPPORTED = 5
};

enum MkbhDtype { MKBH_BF16 = 0, MKBH_F32 = 1 };       /* weights, activations, keys and values */
enum MkbhMixer { MKBH_DELTA_RULE = 0, MKBH_DIFF_ATTENTION = 1, MKBH_ATTENTION = 2, MKBH_LATENT_ATTENTION = 3 };
enum MkbhNorm { MKBH_LAYER_NORM = 0, MKBH_RMS_NORM = 1 };
enum MkbhFeedForward { MKBH_POLY_NORM = 0, MKBH_CLAMPED_GLU = 1 };

/* Opcodes of the decode instruction set (word 0 of a 32-word instruction; 0 is a no-op).
 * Word 1 is the layer, words 2.. are listed. */
enum MkbhOpcode {
    MKBH_OP_NOOP = 0,
    MKBH_OP_NORM_PROJ = 1,   /* row_start, row_end: norm, input convolution, stacked input projection, convolution */
    MKBH_OP_DELTA_STEP = 2,  /* head, col_start, col_end: one step of the recurrence */
    MKBH_OP_ATTENTION = 3,   /* kv_head (latent: group of heads), split, num_splits */
    MKBH_OP_OUT_PROJ = 4,    /* row_start, row_end: output projection, layer scale, residual */
    MKBH_OP_NORM_UP = 5,     /* row_start, row_end: norm, up projection (gated: the unit as well) */
    MKBH_OP_DOWN = 6,        /* row_start, row_end: activation, down projection, scale, residual (beside a mixer: aside) */
    MKBH_OP_HEAD = 7,        /* row_start, row_end: final norm, logits, argmax */
    MKBH_OP_ENTER = 8,       /* row_start, row_end: x <- W [x; embedding] before a pass of the loop */
    MKBH_OP_ABSORB = 9,      /* row_start, row_end (of one head): query times the key up-projection */
    MKBH_OP_EXPAND = 10      /* row_start, row_end (of one head), num_splits: latent output to value space */
};

#define MKBH_INTS_PER_INSTRUCTION 32
#define MKBH_TIMING_SLOTS 128
#define MKBH_STATUS_WORDS 16
/* columns of the per-layer barrier row: one arrival counter per phase of the layer (by opcode) */
#define MKBH_BARRIERS_PER_LAYER 12
#define MKBH_FLAG_RECORD_TIMINGS 1u

/* Matrices are row-major [out, in] in the model dtype with `in` padded with zeros to a multiple
 * of 8 elements; vectors and biases are float. */
typedef struct MkbhLayer {
    int32_t mixer;             /* MkbhMixer */
    int32_t heads, kv_heads;   /* delta rule: heads only; latent: kv_heads = groups of heads in a decode step */
    int32_t dim, vdim;         /* delta rule: dim only; latent: dim = unrotated query/key dimensions */
    int32_t rank;              /* delta rule: inner size of the low-rank decay; latent: size of the latent */
    int32_t window, keep_first;
    int32_t owns_kv;           /* attention: 0 when it reads another layer's keys and values */
    int32_t cache_keep;        /* rows that hold positions 0..cache_keep-1 */
    int32_t cache_ring;        /* rows that hold later positions, modulo */
    int32_t ff;                /* 0: no feed-forward */
    int32_t in_rows;           /* rows of in_w: delta [r k v a g w1], differential [q g (k v)],
                                  attention [q k v], latent [q (head: dim, rot_dim) | latent | rotated key] */
    int32_t chunk;             /* attention: only keys of the query's own chunk; 0: window */
    int32_t ff_kind;           /* MkbhFeedForward; the rows of a gated up_w alternate gate, up */
    int32_t parallel;          /* the feed-forward reads the mixer's input stream, both are added at once */
    int32_t x_buf;             /* decode: which of the two residual buffers the layer works on */
    int32_t canon_taps;        /* taps of the convolution on the mixer's input (0: none) */
    int32_t conv_taps;         /* taps of the convolution on the stacked projection (0: none) */
    int32_t rot_dim;           /* latent: rotated query/key dimensions */
    int32_t rope_dims;         /* rotated dimensions of `rope` */
    float scale, diff, lambda;
    float decay_scale, unit_eps;
    float act[4];              /* PolyNorm coefficients */
    float glu_limit, glu_alpha;
    const void *in_w, *out_w, *up_w, *down_w;
    const float *in_bias;      /* [in_rows] or NULL */
    const float *norm1, *norm2;
    const float *ls1, *ls2;    /* layer scales, or NULL */
    const void *decay_w2;      /* [heads*dim, rank], model dtype, not padded */
    const float *decay_w0;     /* [heads*dim] */
    const float *out_norm;     /* [heads*dim] */
    /* Rows are positions (cache_keep + cache_ring of them).  Differential: [slots, rows, kv_heads, 2, dim]
     * and [slots, rows, kv_heads, vdim].  Rotary: [slots, kv_heads, rows, dim] and [slots, kv_heads, rows,
     * vdim].  Latent: [slots, rows, pad8(rank) + pad8(rot_dim), plus 8 if that is an even number of
     * eights], the latent, then the rotated key. */
    void *k_cache, *v_cache;
    float *state;              /* [slots, heads, dim (value channel), dim (key channel)] */
    const void *enter_w;       /* [width, pad8(2 width)]: the run starts a pass of the loop; else NULL */
    /* Convolutions over time: inputs of the last taps-1 positions in a ring by position, and the
     * sum of their terms for the next position. */
    const float *canon_w;      /* [canon_taps, width] */
    const float *canon_gain;   /* [width]: norm1 * (1 + last tap) */
    float *canon_hist;         /* [slots, canon_taps - 1, width] */
    float *canon_part;         /* [slots, 2 (position parity), width] */
    const float *conv_w;       /* [conv_taps, in_rows] */
    float *conv_hist;          /* [slots, conv_taps - 1, in_rows] */
    float *conv_part;          /* [slots, in_rows] */
    const float *q_norm, *k_norm; /* [dim]; latent: k_norm [rank] */
    const float *temp, *sink;  /* [heads] */
    const float *rope;         /* [max_positions, rope_dims / 2, 2]: cosine, sine of neighbours' angles */
    const float *value_rope;   /* [max_positions, vdim / 2, 2]: values turn with it, outputs back; or NULL */
    const void *absorb_w;      /* latent: [heads * rank, pad8(dim)] */
    const void *expand_w;      /* latent: [heads * (dim + vdim), pad8(rank)]: keys of all heads, values of all heads */
} MkbhLayer;

typedef struct MkbhGlobals {
    uint32_t abi_version, struct_bytes;
    int32_t dtype;             /* MkbhDtype */
    int32_t num_layers, width, vocab, max_positions, slots;
    int32_t norm_kind, reserved; /* MkbhNorm */
    float eps, embed_scale;
    const void *embed;         /* [vocab, width], not padded */
    const void *pos;           /* [max_positions, width], not padded; or NULL */
    const void *head;          /* [vocab, pad8(width)] */
    const float *final_norm;
    const MkbhLayer *layers_host;
    const MkbhLayer *layers_device;

    /* the token(s) */
    const int32_t *tokens;     /* device: decode reads tokens[0] */
    int32_t num_tokens;        /* prefill */
    int32_t slot;
    int32_t pos0;              /* position of the first token */
    const int32_t *pos_device; /* decode: overrides pos0 when set */
    const int32_t *want_rows;  /* device, prefill: rows of the portion whose logits are wanted */
    int32_t num_want;
    float *logits;             /* [num_want, vocab] (decode: [vocab]) */
    int32_t *argmax_out;       /* decode: argmax of the logits (smallest index among equals); may be NULL */
    float *layers_out;         /* prefill: NULL or [num_layers, num_tokens, width], the residual stream after every layer */

    /* decode buffers */
    int32_t *counters;         /* 2 words (running argmax), [num_layers + 1, MKBH_BARRIERS_PER_LAYER], then
                                  [num_layers, max kv_heads]; 8-byte aligned, zeroed by the library before every launch */
    int32_t num_counters, max_kv_heads;
    const int32_t *instructions; /* [num_sms, queue_len, 32] */
    int32_t *timings;          /* [num_sms, queue_len, 128] or NULL */
    int32_t num_sms, queue_len;
    const int32_t *arrivals;   /* device [num_layers + 1, MKBH_BARRIERS_PER_LAYER]: instructions per phase */
    float *attn_part;          /* [max heads, 2, max_splits, 4 + part_vdim rounded up to 4] */
    int32_t max_splits, part_vdim; /* largest split count and vdim of any attention layer */

    /* activations: x [rows, width]; proj [rows, max in_rows, ff]; act [rows, ld] in the model dtype;
     * mixed [rows, widest mixer output]; decay [rows, max of heads*dim + 2*heads of a recurrence] */
    float *x, *proj, *mixed, *decay; /* (decode: x is two rows) */
    void *act;
    int64_t x_elems, proj_elems, mixed_elems, act_elems, decay_elems; /* capacities, checked before launching */
    /* parallel layers, convolutions, rotary and latent attention (NULL without them).
     * Prefill, model dtype: query [rows, widest heads * (dim + rot_dim)], act2 [rows, width],
     * ffn [rows, ff], keys [max_positions, widest heads * (dim + vdim)]; tail: float [taps, width].
     * Decode, float: side [ff | width | heads * rank]. */
    void *query, *act2, *ffn, *keys;
    float *tail, *side;
    int64_t query_elems, act2_elems, ffn_elems, keys_elems, tail_elems, side_elems;
    int32_t side_ff, side_rank;  /* room of the first and the third part of `side` */
    int32_t portion_capacity, reserved2;

    uint32_t flags;
    uint32_t wait_timeout_ms;  /* 0: 2000 */
    int32_t *status;           /* device, MKBH_STATUS_WORDS int32 */
} MkbhGlobals;

int mkb_hybrid_decode(const MkbhGlobals *g, void *cuda_stream);
int mkb_hybrid_prefill(const MkbhGlobals *g, void *cuda_stream);
/* Synchronise and read the status record (code, sm, instruction, opcode, role, detail[4], ...). */
int mkb_hybrid_sync_status(const MkbhGlobals *g, void *cuda_stream, int32_t out[MKBH_STATUS_WORDS]);
/* Check a host copy of the instruction tensor against the shapes in `g`. */
int mkb_hybrid_validate(const MkbhGlobals *g, const int32_t *host_instructions);
const char *mkb_hybrid_last_error(void);
int mkb_hybrid_abi_version(void);
size_t mkb_hybrid_layer_bytes(void);
size_t mkb_hybrid_globals_bytes(void);

#ifdef __cplusplus
}
#endif
#endif /* MKB200_HYBRID_H */
