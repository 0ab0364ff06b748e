/*
 * megaqwen_hybrid — C ABI of the layer-listed decoder: a model whose layers are given one by one, each with a
 * mixer (lightning attention or latent attention), an optional gated feed-forward beside it, and a stretch of
 * layers that may run several times in a row with the same weights (design "Satosun").
 *
 * Conventions are those of megaqwen_b200.h: the caller owns every buffer, token and position are DEVICE scalars
 * (so that steps chain without a host round trip and can be captured in a CUDA graph), calls are asynchronous on
 * the given stream and return 0, a negative MQ_ERR_* code or a positive cudaError_t.  Status bits and launch
 * flags are shared with that header.
 *
 * Every size is a run-time value.  Sizes below are PADDED sizes: width, heads' dim / rot / vdim, rank and ff are
 * rounded up to multiples of 16 by the packer, the padding of every weight and norm holds zeros, and so does the
 * padding of every activation.  The element counts that a norm averages over are given separately.
 */
#ifndef MEGAQWEN_HYBRID_H
#define MEGAQWEN_HYBRID_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* Type of weights, activations and the latent cache.  Residual stream, norms, scores, recurrent state and logits
 * are 32-bit in both; with MQH_F32 the matrix products are 32-bit as well. */
#define MQH_BF16 0
#define MQH_F32 1

/* Mixers. */
#define MQH_LIGHTNING 0
#define MQH_LATENT 1

#define MQH_CHUNK 128      /* tokens of one chunk of the chunked recurrence; decay_pow holds MQH_CHUNK + 1 powers */
#define MQH_SEGMENT 32     /* every segment of w_in / w_ukv starts at a multiple of this many rows */

/* One layer.  w_in is the projection of the normalised input, its row segments in this order, each padded with
 * zero rows to a multiple of MQH_SEGMENT:
 *   lightning  q [heads*dim] | k [heads*dim] | v [heads*vdim] | g [heads*vdim] | gate, up interleaved [2 ff]
 *   latent     q unrotated [heads*dim] | q rotated [heads*rot] | latent, shared rotated key [rank + rot] |
 *              gate, up interleaved [2 ff]
 * (ff = 0: no feed-forward, no segment).  w_out [width, heads*vdim + ff] is the output projection of the mixer
 * beside the down projection: one product adds both to the residual stream. */
typedef struct MqhLayer {
    int kind;
    int heads, dim, vdim;
    int rank, rot;            /* latent */
    int ff;
    int mix_norm_n;           /* elements of the mixer's own norm, without padding */
    float scale;              /* latent: score scale */
    const float* norm;        /* [width] gain of the layer's norm (1 + stored weight) */
    const void* w_in;
    const void* w_out;
    const float* mix_norm;    /* lightning [heads*vdim], latent [rank] */
    const float* decay_pow;   /* lightning [heads, MQH_CHUNK + 1]: decay^0, decay^1, .. */
    const void* w_ukv;        /* latent: keys [heads*dim] | values [heads*vdim] (segments), each row [rank] */
    const void* w_uk_t;       /* latent [heads*rank, dim]: W_uk of every head transposed */
    const float* sink;        /* latent [heads] */
    const float* rope;        /* latent [max_seq, rot/2, 2]: cos, sin of position * frequency */
} MqhLayer;

typedef struct MqhModel {
    int dtype;
    int width, norm_n;        /* padded width, elements of a norm over the width */
    int vocab, max_seq;
    float embed_scale, eps, residual_mult;
    int num_layers;
    int loop_start, loop_stop, loop_times;   /* loop_times = 0: no loop */
    const MqhLayer* layers;   /* HOST array */
    const void* w_loop;       /* [width, 2 width] on [x; embedding output], or null without a loop */
    const void* embed;        /* [vocab, width] */
    const float* final_norm;  /* [width] gain */
    const void* head;         /* [vocab, width] */
} MqhModel;

typedef struct MqhBuffers {
    void* workspace;          /* mqh_workspace_bytes, zeroed once by the caller, 256-byte aligned */
    size_t workspace_bytes;
    int max_tokens;           /* most tokens of one prefill call */
    void* const* run_state;   /* HOST array of mqh_run_count device pointers, mqh_state_bytes each, 256-byte aligned */
    unsigned int* status;     /* u32 [1], sticky MQ_STATUS_* bits */
} MqhBuffers;

/* Layer runs of one forward pass (a looped layer counts each time), the layer of a run (or -1), and the bytes of
 * cache or recurrent state that the run owns.  A recurrent state (mqh_state_recurrent = 1) starts a sequence as
 * zeros; a cache may hold anything. */
int mqh_run_count(const MqhModel* model);
int mqh_run_layer(const MqhModel* model, int run);
size_t mqh_state_bytes(const MqhModel* model, int run);
int mqh_state_recurrent(const MqhModel* model, int run);

/* Rows of w_in and w_ukv (segments with their padding); checks of the packer. */
int mqh_in_rows(const MqhLayer* layer);
int mqh_ukv_rows(const MqhLayer* layer);

size_t mqh_workspace_bytes(const MqhModel* model, int max_tokens);
int mqh_logits_ld(const MqhModel* model);        /* row length of a prefill's logits, >= vocab */
int mqh_decode_launch_count(const MqhModel* model);

/* One greedy decode step, as mq_launch_decode: reads *in_token and *position, updates cache and state, writes the
 * arg-max token (lowest index among equals) to *out_token and, if logits != NULL, the logits as fp32 [vocab]. */
int mqh_launch_decode(const MqhModel* model, const MqhBuffers* buf, const int* in_token, int* out_token, const int* position, float* logits,
                      int flags, void* stream);

/* n tokens that continue the sequence at pos0 (a whole prompt or a portion of one).  *out_token is the token that
 * follows the last one.  want_rows: device array of n_want row numbers (0 .. n - 1) whose logits are written to
 * logits [n_want, mqh_logits_ld]; null with n_want = 0.  launches (may be null) receives the kernels launched. */
int mqh_launch_prefill(const MqhModel* model, const MqhBuffers* buf, const int* ids, int n, int pos0, const int* want_rows, int n_want,
                       int* out_token, float* logits, int* launches, void* stream);

/* The mechanisms on their own, each with the kernels of the two entry points above.
 * mqh_launch_lightning: q, k [n, heads*dim], v [n, heads*vdim] (after their activation), state [heads, dim, vdim]
 * fp32 in and out, o [n, heads*vdim] fp32.  chunked = 0: token after token, 1: in chunks (bf16 only). */
size_t mqh_lightning_scratch_bytes(int n, int heads, int dim, int vdim);
int mqh_launch_lightning(int dtype, const void* q, const void* k, const void* v, const float* decay_pow, float* state, float* o, int n, int heads,
                         int dim, int vdim, int chunked, void* scratch, void* stream);
/* mqh_launch_causal_attention: q [n, heads*dim], q_rot [n, heads*rot], k [pos0 + n, heads*dim], k_rot [pos0 + n, rot] with row length
 * ld_rot, v [pos0 + n, heads*vdim] -> out [n, heads*vdim]; sink [heads] fp32 or null.  tensor_cores = 1: tcgen05 (bf16 only). */
int mqh_launch_causal_attention(int dtype, const void* q, const void* q_rot, const void* k, const void* k_rot, int ld_rot, const void* v,
                                const float* sink, void* out, int n, int pos0, int heads, int dim, int rot, int vdim, float scale,
                                int tensor_cores, unsigned int* status, void* stream);

/* Shared with megaqwen_b200.h (the same code in both libraries). */
int mq_launch_fill_iota(int* dst, int start, int n, void* stream);
int mq_launch_find_first_eos(const int* tokens, int n, const int* eos_ids, int n_eos, int* out_index, void* stream);

#ifdef __cplusplus
}
#endif
#endif
