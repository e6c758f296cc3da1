/*
 * twm_dense.h — decoder-only models with 16-bit or 32-bit dense weights: one step of a sequence
 * (a portion of its prompt, or one decoded token) over per-sequence state kept in slots.
 *
 * A model is a list of layer runs (a layer that runs several times appears several times, with the same
 * weights and state of its own).  A layer is a mixer and an optional feed-forward, each with an optional RMS
 * norm of its input and of its OUTPUT, which joins the FP32 residual stream.  The mixers:
 *   TWM_MIX_SIGMOID  token shift, fused q|k|v|gate projection, q/k norm over the whole row, windowed sigmoid
 *                    attention with kept first keys and a per-head distance bias, output gate
 *   TWM_MIX_LATENT   windowed softmax attention over keys and values expanded from one normed latent per token,
 *                    with a rotated key part shared by all heads and one output gate per head
 *   TWM_MIX_GLA      gated linear attention: a matrix state per head with one decay per key channel, per-head
 *                    norm, silu gate
 * The feed-forwards: gated (gelu_tanh(gate) * up), or routed (the sum of the chosen experts' outputs times
 * their softmax scores, experts W_down relu(W_up h)^2).  Every part is switched by its pointer or size: a
 * NULL shift, q_norm, norm1, pre1 ... leaves that mechanism out.
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
enum { TWM_MIX_SIGMOID = 0, TWM_MIX_LATENT = 1, TWM_MIX_GLA = 2 };

typedef struct twm_dense_layer {
    int mixer;                   /* TWM_MIX_* */
    int heads, kv_heads;         /* query head h reads key/value head h / (heads / kv_heads) */
    int dim, vdim;               /* per-head query/key and value sizes */
    int dim_pad, vdim_pad;       /* the same as laid out in memory */
    int window;                  /* position i sees j <= i with i - j < window ... */
    int keep_first;              /* ... or j < keep_first */
    int ff_pad;                  /* 0 = the layer has no feed-forward */
    float scale;                 /* factor of q.k (GLA: of q) */
    /* w_in rows, each block of width_pad columns.
     * SIGMOID: heads*dim_pad | kv_heads*dim_pad | kv_heads*vdim_pad | heads*vdim_pad (gate)
     * LATENT:  heads*(dim_pad + rot_pad) | rank_pad (latent) | rot_pad (shared key part) | heads (gate) up to a multiple of 16
     * GLA:     heads*dim_pad | heads*dim_pad | heads*vdim_pad | heads*vdim_pad (gate) | rank_pad (low-rank) */
    const void* w_in;
    const void* w_out;           /* [width][heads*vdim_pad] */
    const void* w_gate_up;       /* gated: [ff_pad | ff_pad][width_pad]; routed: [experts][ff_pad][width_pad] */
    const void* w_down;          /* gated: [width][ff_pad]; routed: [experts][width][ff_pad] */
    const float* q_norm;         /* [heads*dim_pad] or NULL */
    const float* k_norm;         /* [kv_heads*dim_pad] or NULL */
    const float* bias_table;     /* [heads][bias_len]: added to the scaled score at distance d; NULL = 0 */
    const float* shift;          /* [width_pad] token-shift factors or NULL */
    const float* norm1;          /* [width_pad] weights of the norm on the mixer's output */
    const float* norm2;          /* [width_pad] ... on the feed-forward's output */
    const float* pre1;           /* [width_pad] ... on the mixer's input, or NULL; not together with shift */
    const float* pre2;           /* [width_pad] ... on the feed-forward's input, or NULL */
    const float* step;           /* [width_pad] added to the residual stream ahead of this run, or NULL */
    /* LATENT, and rank / rank_pad of GLA's low-rank projection */
    int rank, rank_pad;          /* size of the latent */
    int rot_pad;                 /* rotated part of a query and of the shared key part: pairs of neighbours */
    const void* w_expand;        /* [heads*dim_pad | heads*vdim_pad][rank_pad]: keys and values from the latent */
    const float* latent_norm;    /* [rank_pad] */
    const float* rot_table;      /* [capacity][rot_pad/2][2]: cosine and sine at every position */
    void* latent_cache;          /* [slots][capacity][rank_pad + rot_pad] */
    /* GLA */
    float inv_tau;               /* log decay = log(sigmoid(z)) * inv_tau */
    const void* w_decay;         /* [heads*dim_pad][rank_pad] */
    const float* decay_bias;     /* [heads*dim_pad] */
    const float* head_norm;      /* [vdim_pad] */
    float* gla_state;            /* [slots][heads][dim_pad][vdim_pad] */
    /* routed feed-forward: experts > 0 */
    int experts, top;            /* experts a token uses */
    int groups, keep;            /* experts of the `keep` best of `groups` groups of neighbours can be chosen */
    const void* w_router;        /* [experts][width_pad] */
    void* k_cache;               /* [slots][capacity][kv_heads*dim_pad] */
    void* v_cache;               /* [slots][capacity][kv_heads*vdim_pad] */
    float* shift_state;          /* [slots][2][width_pad]: the previous token's mixer input, by parity of its position */
} twm_dense_layer;

typedef struct twm_dense_model {
    int dtype;                   /* TWM_DENSE_BF16 or TWM_DENSE_F32: weights, caches and matrix-product inputs */
    int width, width_pad, vocab;
    int n_layers;                /* layer runs */
    int bias_len;                /* entries per head of the bias tables; > every distance that can occur */
    int capacity;                /* tokens per slot */
    int slots;
    float eps;
    float embed_scale;           /* factor of the embedding's rows */
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
    void* act;                   /* [max_rows][widest ff_pad], routed: [max_rows * top][ff_pad] */
    float* vec;                  /* decode: [widest w_in + widest heads*vdim_pad + widest act (routed: top*ff_pad) + width_pad] */
    float* logits;               /* [max_want][vocab] */
    /* LATENT (NULL without): the tokens a step's queries can see, at most max_keys */
    int max_keys;
    void* lat;                   /* [max_keys][widest rank_pad + rot_pad] */
    void* kv;                    /* [max_keys][widest heads*(dim_pad + vdim_pad)] */
    /* GLA (NULL without) */
    float* decay;                /* [max_rows][widest heads*dim_pad] */
    float* chunk_state;          /* [(max_rows + 63) / 64][widest heads*dim_pad*vdim_pad] */
    float* mix;                  /* [max_rows][widest heads*vdim_pad] */
    /* routed (NULL without) */
    float* router_logits;        /* [max_rows][widest experts] */
    int* route;                  /* [3][max_rows * widest top] choices, their places, their rows; then [2 * widest experts + 1] counts, offsets */
    float* route_weight;         /* [max_rows * widest top] */
    void* grouped;               /* [max_rows * widest top][width_pad] */
    void* expert_out;            /* [max_rows * widest top][width_pad] */
    int max_slots;               /* max_rows * widest top */
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
enum { TWM_EPI_STORE = 0, TWM_EPI_STORE_F32 = 1, TWM_EPI_GELU_GLU = 2, TWM_EPI_RELU2 = 3 };
/* C[M][N] = A[M][K] . W[N][K]^T with FP32 accumulation.  GELU_GLU: W is [N | N][K] (gate, up), C = gelu_tanh(gate) * up.
 * C has the input type except for STORE_F32.  kernel: 0 = chosen by size, 1 = plain tiles, 2 = tcgen05, 64/128/256 = tcgen05 with
 * tiles of that many columns, 512 = tiles of 256 x 256 on a pair of SMs. */
twm_status twm_dense_gemm(int dtype, const void* a, int lda, const void* w, int ldw, void* c, int ldc, int M, int N, int K,
                          int epilogue, int kernel, int flags, void* stream);
/* Choices (ids, weights: [rows][top]) of `rows` tokens by their router logits [rows][experts]. */
twm_status twm_dense_route(const float* logits, int experts, int top, int groups, int keep, int rows, int* ids, float* weights, int flags,
                           void* stream);
/* C[r] = epi(A[r] . W[e]^T) for the rows offsets[e] <= r < offsets[e + 1] of every expert e (device array of experts + 1, ending at
 * `rows`); W [experts][N][ldw].  Epilogues STORE, STORE_F32, RELU2; kernels 0, 1, 2, 64, 128, 256 of twm_dense_gemm. */
twm_status twm_dense_grouped_gemm(int dtype, const void* a, int lda, const void* w, int ldw, void* c, int ldc, const int* offsets, int experts,
                                  int rows, int N, int K, int epilogue, int kernel, int flags, void* stream);
/* The GLA mixer of `rows` tokens between its projections: buffers->proj as the fused projection leaves it, buffers->att out.
 * kernel: 0 = by size, 1 = token by token, 2 = chunks. */
twm_status twm_dense_gla(const twm_dense_model* m, int layer, const twm_dense_buffers* b, int rows, int kernel, int flags, void* stream);
/* Attention of `rows` queries at positions meta[0] ... over the slot's cache (already holding their keys and values);
 * proj rows as the fused projection leaves them (q normalised in place, gate = last block).  kernel: 0 = by size,
 * 1 = one query per CTA, 2 = warp-level tensor-core tiles (SIGMOID), 3 = tcgen05 tiles.  LATENT: norms, rotates and expands the
 * step's latents first (proj as the fused projection leaves it). */
twm_status twm_dense_attention(const twm_dense_model* m, int layer, const twm_dense_buffers* b, int rows, int first_pos,
                               int kernel, int flags, void* stream);

twm_status twm_dense_device_error(void* stream, unsigned int* word);
const char* twm_dense_status_string(int s);
const char* twm_dense_last_error(void);

#ifdef __cplusplus
}
#endif
#endif /* TWM_DENSE_H */
