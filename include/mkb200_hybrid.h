/*
 * C ABI of libmkb200_hybrid.so: decoders whose layers are listed one by one, each with a
 * recurrent (generalized delta rule) or a windowed-attention mixer and an optional
 * feed-forward.  Plain pointers and sizes; no framework type crosses it.
 *
 * Two entry points do the work, both asynchronous on the given stream:
 *   mkb_hybrid_decode   one token of one sequence, ONE persistent kernel launch that
 *                       interprets per-SM instruction queues (as mkb_launch does);
 *   mkb_hybrid_prefill  a portion of 1..portion_capacity tokens of one sequence, a sequence
 *                       of tensor-core / scan / attention kernels.
 * Both read and advance the same per-slot state (key/value rows, recurrent matrices), so a
 * sequence may be cut into portions and single tokens in any way.
 */
#ifndef MKB200_HYBRID_H
#define MKB200_HYBRID_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define MKBH_ABI_VERSION 1

enum MkbhCode { /* same values as MkbCode of mkb200.h */
    MKBH_OK = 0,
    MKBH_ERR_INVALID_ARGUMENT = 1,
    MKBH_ERR_CUDA = 2,
    MKBH_ERR_DEVICE_TIMEOUT = 3,
    MKBH_ERR_BAD_OPCODE = 4,
    MKBH_ERR_UNSUPPORTED = 5
};

enum MkbhDtype { MKBH_BF16 = 0, MKBH_F32 = 1 };       /* weights, activations, keys and values */
enum MkbhMixer { MKBH_DELTA_RULE = 0, MKBH_DIFF_ATTENTION = 1 };

/* Opcodes of the decode instruction set (word 0 of a 32-word instruction; 0 is a no-op).
 * Word 1 is the layer, words 2.. are listed. */
enum MkbhOpcode {
    MKBH_OP_NOOP = 0,
    MKBH_OP_NORM_PROJ = 1,   /* row_start, row_end: layer norm, stacked input projection */
    MKBH_OP_DELTA_STEP = 2,  /* head, col_start, col_end: one step of the recurrence */
    MKBH_OP_ATTENTION = 3,   /* kv_head, split, num_splits: windowed differential attention */
    MKBH_OP_OUT_PROJ = 4,    /* row_start, row_end: output projection, layer scale, residual */
    MKBH_OP_NORM_UP = 5,     /* row_start, row_end: layer norm, up projection */
    MKBH_OP_DOWN = 6,        /* row_start, row_end: PolyNorm, down projection, scale, residual */
    MKBH_OP_HEAD = 7         /* row_start, row_end: final norm, logits, argmax */
};

#define MKBH_INTS_PER_INSTRUCTION 32
#define MKBH_TIMING_SLOTS 128
#define MKBH_STATUS_WORDS 16
/* columns of the per-layer barrier row: one arrival counter per phase of the layer (by opcode) */
#define MKBH_BARRIERS_PER_LAYER 8
#define MKBH_FLAG_RECORD_TIMINGS 1u

/* Matrices are row-major [out, in] in the model dtype with `in` padded with zeros to a multiple
 * of 8 elements; vectors and biases are float. */
typedef struct MkbhLayer {
    int32_t mixer;             /* MkbhMixer */
    int32_t heads, kv_heads;   /* delta rule: heads only */
    int32_t dim, vdim;         /* delta rule: dim only */
    int32_t rank;              /* delta rule: inner size of the low-rank decay */
    int32_t window, keep_first;
    int32_t owns_kv;           /* attention: 0 when it reads another layer's keys and values */
    int32_t cache_keep;        /* rows that hold positions 0..cache_keep-1 */
    int32_t cache_ring;        /* rows that hold later positions, modulo */
    int32_t ff;                /* 0: no feed-forward */
    int32_t in_rows;           /* rows of in_w: delta [r k v a g w1], attention [q g (k v)] */
    float scale, diff, lambda;
    float decay_scale, unit_eps;
    float act[4];              /* PolyNorm coefficients */
    const void *in_w, *out_w, *up_w, *down_w;
    const float *in_bias;      /* [in_rows] or NULL */
    const float *norm1, *norm2, *ls1, *ls2;
    const void *decay_w2;      /* [heads*dim, rank], model dtype, not padded */
    const float *decay_w0;     /* [heads*dim] */
    const float *out_norm;     /* [heads*dim] */
    void *k_cache;             /* [slots, cache_keep + cache_ring, kv_heads, 2, dim] */
    void *v_cache;             /* [slots, cache_keep + cache_ring, kv_heads, vdim] */
    float *state;              /* [slots, heads, dim (value channel), dim (key channel)] */
} MkbhLayer;

typedef struct MkbhGlobals {
    uint32_t abi_version, struct_bytes;
    int32_t dtype;             /* MkbhDtype */
    int32_t num_layers, width, vocab, max_positions, slots;
    float eps, embed_scale;
    const void *embed;         /* [vocab, width], not padded */
    const void *pos;           /* [max_positions, width], not padded */
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
    float *attn_part;          /* [max heads, 2, max_splits, part_vdim + 2] */
    int32_t max_splits, part_vdim; /* largest split count and vdim of any attention layer */

    /* activations: x [rows, width]; proj [rows, max in_rows, ff]; act [rows, ld] in the model dtype;
     * mixed [rows, widest mixer output]; decay [rows, max of heads*dim + 2*heads of a recurrence] */
    float *x, *proj, *mixed, *decay;
    void *act;
    int64_t x_elems, proj_elems, mixed_elems, act_elems, decay_elems; /* capacities, checked before launching */
    int32_t portion_capacity;

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
