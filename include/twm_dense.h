/*
 * twm_dense.h — decoder-only models with 16-bit or 32-bit dense weights: one step of a sequence
 * (a portion of its prompt, or one decoded token) over per-sequence state kept in slots.
 *
 * A model is a list of layers; a layer is a mixer (token shift, fused q|k|v|gate projection,
 * q/k norm over the whole row, windowed attention with kept first keys and a per-head distance
 * bias, output gate, output projection) and an optional gated feed-forward, each followed by an
 * RMS norm of its OUTPUT that joins the FP32 residual stream.  Every part is switched by its
 * pointer or size: a NULL shift, q_norm, norm1 ... leaves that mechanism out.
 *
 * Same conventions as twmarlin.h: device pointers owned by the caller, enqueue only, nothing
 * allocated, status returned.  Position and slot are read from device memory (buffers->meta), so a
 * captured decode step serves every position and slot.
 *
 * Padding.  Every row length a kernel walks is padded by the loader to a multiple of 16 elements
 * (width_pad, dim_pad, vdim_pad, ff_pad) with zero weights, so padded activations are exactly zero.
 */
#ifndef TWM_DENSE_H
#define TWM_DENSE_H

#include "twmarlin.h"

#ifdef __cplusplus
extern "C" {
#endif

enum { TWM_DENSE_F32 = 0, TWM_DENSE_BF16 = 2 };

typedef struct twm_dense_layer {
    int heads, kv_heads;         /* query head h reads key/value head h / (heads / kv_heads) */
    int dim, vdim;               /* per-head query/key and value sizes */
    int dim_pad, vdim_pad;       /* the same as laid out in memory */
    int window;                  /* position i sees j <= i with i - j < window ... */
    int keep_first;              /* ... or j < keep_first */
    int ff_pad;                  /* 0 = the layer has no feed-forward */
    float scale;                 /* factor of q.k */
    const void* w_in;            /* [heads*dim_pad | kv_heads*dim_pad | kv_heads*vdim_pad | heads*vdim_pad][width_pad] */
    const void* w_out;           /* [width][heads*vdim_pad] */
    const void* w_gate_up;       /* [ff_pad | ff_pad][width_pad] */
    const void* w_down;          /* [width][ff_pad] */
    const float* q_norm;         /* [heads*dim_pad] or NULL */
    const float* k_norm;         /* [kv_heads*dim_pad] or NULL */
    const float* bias_table;     /* [heads][bias_len]: added to the scaled score at distance d; NULL = 0 */
    const float* shift;          /* [width_pad] token-shift factors or NULL */
    const float* norm1;          /* [width_pad] weights of the norm on the mixer's output */
    const float* norm2;          /* [width_pad] ... on the feed-forward's output */
    void* k_cache;               /* [slots][capacity][kv_heads*dim_pad] */
    void* v_cache;               /* [slots][capacity][kv_heads*vdim_pad] */
    float* shift_state;          /* [slots][2][width_pad]: the previous token's mixer input, by parity of its position */
} twm_dense_layer;

typedef struct twm_dense_model {
    int dtype;                   /* TWM_DENSE_BF16 or TWM_DENSE_F32: weights, caches and matrix-product inputs */
    int width, width_pad, vocab, n_layers;
    int bias_len;                /* entries per head of the bias tables; > every distance that can occur */
    int capacity;                /* tokens per slot */
    int slots;
    float eps;
    const void* embed;           /* [vocab][width_pad] */
    const void* pos_embed;       /* [>= capacity][width_pad] or NULL */
    const void* head;            /* [vocab][width_pad] */
    const float* final_norm;     /* [width_pad] */
    const twm_dense_layer* layers;   /* host array */
} twm_dense_model;

/* Scratch of one step, allocated once and ZEROED by the caller (padding columns stay zero). */
typedef struct twm_dense_buffers {
    int max_rows;                /* tokens per step at most */
    int max_want;                /* rows of logits per step at most */
    int* meta;                   /* [0] position of the step's first token, [1] slot, [2] position + 1, [3] decode step counter */
    int* tokens;                 /* [max_rows] */
    int* want;                   /* [max_want] rows whose logits are wanted */
    float* x0;                   /* [max_rows][width_pad] residual stream, two copies used in turn */
    float* x1;
    float* y;                    /* [max_rows][width_pad] a sublayer's output */
    void* a;                     /* [max_rows][width_pad] matrix-product input */
    void* proj;                  /* [max_rows][widest w_in] */
    void* att;                   /* [max_rows][widest heads*vdim_pad] */
    void* act;                   /* [max_rows][widest ff_pad] */
    float* vec;                  /* decode: [widest w_in + widest heads*vdim_pad + widest ff_pad] */
    float* logits;               /* [max_want][vocab] */
} twm_dense_buffers;

/* Enqueue one step of `rows` >= 1 tokens (buffers->tokens) of the sequence in slot meta[1], starting at
 * position meta[0] (= first_pos, which the host passes as well for its bounds checks and launch shapes).
 * The logits of rows want[0 .. n_want) go to buffers->logits [n_want][vocab]; n_want = 0 leaves the head
 * out.  layer_trace, if not NULL: f32 [n_layers][rows][width_pad], the residual stream after every layer. */
twm_status twm_dense_prefill(const twm_dense_model* m, const twm_dense_buffers* b, int rows, int first_pos, int n_want,
                             float* layer_trace, int flags, void* stream);

/* Enqueue one decode step: the token buffers->tokens[0] at position meta[0] of slot meta[1]; nothing about
 * them is a launch parameter.  want_logits != 0: logits to buffers->logits [vocab]. */
twm_status twm_dense_decode(const twm_dense_model* m, const twm_dense_buffers* b, int want_logits, int flags, void* stream);

/* Kernel launches of the last call of this thread to either of the two. */
int twm_dense_launches(void);

/* meta of a step, and tokens[0] unless token < 0: a kernel whose launch parameters carry the values (no host buffer
 * to keep alive). */
twm_status twm_dense_set_step(const twm_dense_buffers* b, int first_pos, int slot, int token, void* stream);

/* Greedy sampling on the device, as twm_argmax_advance: buffers->tokens[0] = argmax(logits[0]) (ties: smallest
 * index), history[meta[3]] = token when it fits, then meta[0], meta[2], meta[3] advance by one. */
size_t twm_dense_argmax_scratch_bytes(void);
twm_status twm_dense_argmax_advance(const twm_dense_buffers* b, int vocab, int row, int* history,
                                    int history_capacity, void* scratch, size_t scratch_bytes, int flags, void* stream);

/* ---- single operations, as the step uses them ---- */
enum { TWM_EPI_STORE = 0, TWM_EPI_STORE_F32 = 1, TWM_EPI_GELU_GLU = 2 };
/* C[M][N] = A[M][K] . W[N][K]^T with FP32 accumulation.  GELU_GLU: W is [N | N][K] (gate, up), C = gelu_tanh(gate) * up.
 * C has the input type except for STORE_F32.  kernel: 0 = chosen by size, 1 = plain tiles, 2 = tcgen05, 64/128/256 = tcgen05 with
 * tiles of that many columns, 512 = tiles of 256 x 256 on a pair of SMs. */
twm_status twm_dense_gemm(int dtype, const void* a, int lda, const void* w, int ldw, void* c, int ldc, int M, int N, int K,
                          int epilogue, int kernel, int flags, void* stream);
/* Attention of `rows` queries at positions meta[0] ... over the slot's cache (already holding their keys and values);
 * proj rows as the fused projection leaves them (q normalised in place, gate = last block).  kernel: 0 = by size,
 * 1 = one query per CTA, 2 = warp-level tensor-core tiles, 3 = tcgen05 tiles. */
twm_status twm_dense_attention(const twm_dense_model* m, int layer, const twm_dense_buffers* b, int rows, int first_pos,
                               int kernel, int flags, void* stream);

twm_status twm_dense_device_error(void* stream, unsigned int* word);
const char* twm_dense_status_string(int s);
const char* twm_dense_last_error(void);

#ifdef __cplusplus
}
#endif
#endif /* TWM_DENSE_H */
