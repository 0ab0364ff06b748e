/*
 * megaqwen_hybrid — C ABI of the layer-listed decoder: a model whose layers are given one by one, each with a
 * mixer (lightning attention, latent attention, gated linear attention, Mamba-2 or grouped-query attention) and an
 * optional gated feed-forward.  Two layer forms exist.  MQH_PARALLEL (design "Satosun"): one norm of the residual
 * stream is read by mixer and feed-forward side by side, and a stretch of layers may run several times in a row with
 * the same weights.  MQH_POST_NORM (design "Vunasun"): mixer and feed-forward follow one another, each reads the
 * residual stream itself, and each result is normed before it is added.
 *
 * Conventions are those of megaqwen_b200.h: the caller owns every buffer, token and position are DEVICE scalars
 * (so that steps chain without a host round trip and can be captured in a CUDA graph), calls are asynchronous on
 * the given stream and return 0, a negative MQ_ERR_* code or a positive cudaError_t.  Status bits and launch
 * flags are shared with that header.
 *
 * Every size is a run-time value.  Sizes below are PADDED sizes unless they say otherwise: width, heads' dim / rot /
 * vdim, rank and ff are rounded up to multiples of 16 by the packer, the padding of every weight and norm holds zeros, and so does the
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
#define MQH_GLA 2          /* state that decays per key channel and token */
#define MQH_MAMBA2 3       /* state that decays per head and token, behind a short convolution */
#define MQH_ATTENTION 4    /* softmax attention over cached keys, heads sharing keys in groups, optionally within chunks */

/* Layer forms. */
#define MQH_PARALLEL 0
#define MQH_POST_NORM 1

#define MQH_CHUNK 128      /* tokens of one chunk of the chunked recurrence; decay_pow holds MQH_CHUNK + 1 powers */
#define MQH_SEGMENT 32     /* every segment of w_in / w_ukv starts at a multiple of this many rows */

/* One layer.  w_in is the projection of the mixer's input, its row segments in this order, each padded with
 * zero rows to a multiple of MQH_SEGMENT:
 *   lightning  q [heads*dim] | k [heads*dim] | v [heads*vdim] | g [heads*vdim]
 *   latent     q unrotated [heads*dim] | q rotated [heads*rot] | latent, shared rotated key [rank + rot]
 *   gla        q [heads*dim] | k [heads*dim] | v [heads*vdim] | g [heads*vdim] | low-rank decay input [rank]
 *   mamba2     z [heads*vdim] | x [heads*vdim] | B [kv_heads*dim] | C [kv_heads*dim] | dt [heads, rounded up to 16]
 *   attention  q [heads*dim] | k [kv_heads*dim] | gate [heads, rounded up to 16]
 * and, in the parallel form with ff > 0, gate and up interleaved [2 ff].  w_out [width, heads*vdim (+ ff)] is the
 * output projection of the mixer; in the parallel form the down projection stands beside it, so that one product
 * adds both to the residual stream.  In the post-norm form the feed-forward has matrices of its own: w_gu (gate and
 * up interleaved, [2 ff rounded up to MQH_SEGMENT, width]) and w_down [width, ff]. */
typedef struct MqhLayer {
    int kind;
    int heads, dim, vdim;     /* mamba2: dim is the state size N */
    int kv_heads;             /* attention: key / value heads; mamba2: groups that share B and C */
    int rank;                 /* latent: width of the latent; gla: inner width of the decay projection */
    int rot;                  /* latent: rotated part (padded); attention: rotated dimensions of a head (exact) */
    int ff;
    int mix_norm_n;           /* elements that share a root mean square in the mixer's own norm (attention: of a head) */
    int norm_parts;           /* lightning 1, gla heads, mamba2 any: parts of the mixer's output norm */
    int vdim_n;               /* vdim without padding */
    int conv;                 /* mamba2: taps */
    int chunk;                /* attention: positions see keys of their own chunk of this many; 0: all before */
    float scale;              /* latent, attention: score scale; gla: factor of q */
    float inv_tau;            /* gla */
    const float* norm;        /* [width] gain: of the input norm, or (post-norm) of the mixer's result, layer scale included */
    const float* norm2;       /* post-norm: [width] gain of the feed-forward's result */
    const void* w_in;
    const void* w_out;
    const void *w_gu, *w_down;   /* post-norm */
    const float* mix_norm;    /* lightning, gla, mamba2 [heads*vdim], latent [rank] */
    const float* decay_pow;   /* lightning [heads, MQH_CHUNK + 1]: decay^0, decay^1, .. */
    const void* w_ukv;        /* latent: keys [heads*dim] | values [heads*vdim] (segments), each row [rank] */
    const void* w_uk_t;       /* latent [heads*rank, dim]: W_uk of every head transposed */
    const float* sink;        /* latent [heads] */
    const float* rope;        /* latent [max_seq, rot/2, 2], attention [max_seq, rot/2, 2]: cos, sin of position * frequency */
    const void* gate_w;       /* gla [heads, rank, dim]: second factor of the decay projection, transposed per head */
    const float* gate_b;      /* gla [heads*dim] */
    const float *conv_w, *conv_b;             /* mamba2 [taps, channels] (the last row is the current token's), [channels] */
    const float *dt_bias, *a_neg, *skip;      /* mamba2 [heads]: bias of dt, -exp(A_log), D */
    const float *q_bias, *k_bias;             /* attention [heads*dim], [kv_heads*dim] */
    const float *q_norm, *k_norm;             /* attention [dim] */
} MqhLayer;

typedef struct MqhModel {
    int dtype;
    int form;                 /* MQH_PARALLEL or MQH_POST_NORM */
    int width, norm_n;        /* padded width, elements of a norm over the width */
    int vocab, max_seq;
    float embed_scale, eps, residual_mult;
    int num_layers;
    int loop_start, loop_stop, loop_times;   /* loop_times = 0: no loop (parallel form only) */
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
int mqh_in_rows(const MqhLayer* layer, int form);
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
size_t mqh_recurrence_scratch_bytes(int n, int heads, int dim, int vdim);
int mqh_launch_lightning(int dtype, const void* q, const void* k, const void* v, const float* decay_pow, float* state, float* o, int n, int heads,
                         int dim, int vdim, int chunked, void* scratch, void* stream);
/* The same for the recurrences whose decay the token sets; layer gives sizes and parameters (kind MQH_GLA or MQH_MAMBA2).
 * q, k [n, kv*dim] with kv = heads (gla) or layer->kv_heads (mamba2), after the convolution; decay_in [n, ld_decay] fp32 is
 * the low-rank input (gla, rank columns) or dt before its bias (mamba2, one column per head). */
int mqh_launch_recurrence(int dtype, const MqhLayer* layer, const void* q, const void* k, const void* v, const float* decay_in, int ld_decay,
                          float* state, float* o, int n, int chunked, void* scratch, void* stream);
/* x [n, channels] -> silu(causal convolution) in y; tokens n at positions pos0 ..; state [taps, channels] in and out, a row per
 * position modulo taps. */
int mqh_launch_conv(int dtype, const void* x, const float* w, const float* b, void* state, void* y, int n, int pos0, int channels, int taps,
                    void* stream);
/* mqh_launch_causal_attention: q [n, heads*dim], q_rot [n, heads*rot], k [pos0 + n, kv_heads*dim], k_rot [pos0 + n, rot] with row length
 * ld_rot, v [pos0 + n, kv_heads*vdim] -> out [n, heads*vdim]; sink [heads] fp32 or null; gate [n, heads] fp32 (before its
 * sigmoid) or null; chunk: see MqhLayer.  rot = 0: no shared key part.  tensor_cores = 1: tcgen05 (bf16 only). */
int mqh_launch_causal_attention(int dtype, const void* q, const void* q_rot, const void* k, const void* k_rot, int ld_rot, const void* v,
                                const float* sink, const float* gate, void* out, int n, int pos0, int heads, int kv_heads, int dim, int rot,
                                int vdim, int chunk, float scale, int tensor_cores, unsigned int* status, void* stream);

/* Shared with megaqwen_b200.h (the same code in both libraries). */
int mq_launch_fill_iota(int* dst, int start, int n, void* stream);
int mq_launch_find_first_eos(const int* tokens, int n, const int* eos_ids, int n_eos, int* out_index, void* stream);

#ifdef __cplusplus
}
#endif
#endif
