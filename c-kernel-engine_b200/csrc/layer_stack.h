/* Decoder models described layer by layer in a config.json: every layer names its token mixer, the mixer's sizes and its feed-forward.
 * layer_stack_config.c reads the description, model_stack_weights.c places the weights, model_stack_mixers.c runs the mixers and
 * model_stack.c the passes. */
#ifndef CKB200_LAYER_STACK_H
#define CKB200_LAYER_STACK_H

#include "linear.h"

enum { STACK_RETENTION = 0, STACK_LATENT_ATTENTION, STACK_CHANNEL_DELTA, STACK_WINDOW_ATTENTION, STACK_LIGHTNING, STACK_WKV };

/* how a layer's norms and sublayers join the residual x:
 *   parallel     h = norm1(x);  x += mixer(h) + ff(h)
 *   output norm  x += norm1(mixer(x));  x += norm2(ff(x)) */
enum { STACK_PARALLEL = 0, STACK_OUTPUT_NORM };

#define STACK_ARMS 2
#define STACK_MIXES 5           /* inputs of wkv: w, r, k, v, g */

/* one token mixer; a layer has one, or two side by side over the same input ("arms") */
typedef struct {
    int type;
    const char *prefix;             /* of its tensors, after "l<i>." */
    /* sizes from the description (those the mixer has) */
    int heads, kv_heads, dim, vdim;
    int taps;                       /* short convolution */
    int q_rank, kv_rank, rot_dim;   /* latent attention */
    int window;                     /* visible positions, 0: all */
    int rot_dims;
    double rot_base;
    double yarn_factor, yarn_fast, yarn_slow, yarn_original;     /* factor 0: no scaling of the rotation */
    float scale;
    float out_scale;                /* on the mixer's result (arms) */
    float *decay_host;              /* [heads] */
    int a_rank, g_rank;             /* low ranks of a decay and an output gate: from the tensors (or the description, synthetic) */

    LinMat uq, ukv, a2, g2;
    int row_q, row_k, row_v, row_g, row_b, row_a1, row_g1, row_dq, row_dkv;    /* first rows inside the layer's `in` */
    int row_uv;                     /* first row of W_uv inside ukv */
    int col;                        /* first column of its output inside the layer's `out` */
    float *head_norm, *q_norm, *kv_norm, *conv_w, *a_log, *dt_bias, *decay, *bonus, *mu, *freq;
    float rot_mul;                  /* on cosines and sines */

    /* per-sequence state: offsets in floats into the model's state (recurrent, previous input), device pointers of caches */
    long long conv_state, rec_state, before;
    void *cache_c, *cache_kr;       /* latent */
    void *cache_k, *cache_v;        /* key/value */
    int cache_cap;                  /* slots per sequence and key head of a key/value cache */
} StackMixer;

typedef struct {
    int arms;
    StackMixer mix[STACK_ARMS];
    int ff;                         /* feed-forward units, 0: none */

    /* weights.  Parallel: one matrix over the normed input (mixer projections, then gate and up), one over [mixer output | ff output].
     * Output norm: the mixer's two, and the feed-forward's two. */
    LinMat in, out, ff_in, ff_out;
    int row_ff;                     /* first gate/up row inside `in` (parallel) or ff_in */
    int z_width;                    /* columns of `in`'s outputs that are kept as fp32 rows */
    int col_ff;                     /* first column of the feed-forward inside `out` (parallel) */
    float *norm1, *norm2;
} StackLayer;

typedef struct {
    int form;
    int tied;                       /* the embedding table is the output projection */
    int width, vocab, n_layers;
    float eps, embed_scale;
    float logit_cap;                /* 0: none */
    StackLayer *layers;
} StackConfig;

/* 0 on success; otherwise an error is recorded and nothing is kept */
int ckb_stack_config_read(const char *path, StackConfig *out);
void ckb_stack_config_free(StackConfig *c);
/* angular steps per position of the rot_dims / 2 pairs, and the factor on cosines and sines */
float ckb_stack_frequencies(const StackMixer *x, float *freq);

#endif
