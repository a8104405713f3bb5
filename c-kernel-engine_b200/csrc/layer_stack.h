/* Decoder models described layer by layer in a config.json: every layer names its token mixer, the mixer's sizes and its feed-forward.
 * layer_stack_config.c reads the description, model_stack.c places the weights and runs the passes. */
#ifndef CKB200_LAYER_STACK_H
#define CKB200_LAYER_STACK_H

#include "linear.h"

enum { STACK_RETENTION = 0, STACK_LATENT_ATTENTION, STACK_CHANNEL_DELTA, STACK_MIXERS };

typedef struct {
    int type;
    /* sizes from the description (those the mixer has) */
    int heads, kv_heads, dim, vdim;
    int taps;                       /* short convolution */
    int q_rank, kv_rank, rot_dim;   /* latent attention */
    int rot_dims;
    double rot_base;
    float scale;
    float *decay_host;              /* [heads] */
    int a_rank, g_rank;             /* low ranks of the delta rule's decay and output gate: from the tensors (or the description, synthetic) */
    int ff;                         /* feed-forward units, 0: none */

    /* weights: one matrix over the normed input (mixer projections, then gate and up), one over [mixer output | ff output] */
    LinMat in, out;
    LinMat uq, ukv, a2, g2;
    int row_q, row_k, row_v, row_g, row_b, row_a1, row_g1, row_dq, row_dkv, row_ff;    /* first rows inside `in` */
    int row_uv;                     /* first row of W_uv inside ukv */
    int z_width;                    /* columns of `in`'s outputs that are kept as fp32 rows */
    int col_ff;                     /* first column of the feed-forward inside `out` */
    float *norm1, *head_norm, *q_norm, *kv_norm, *conv_w, *a_log, *dt_bias, *decay, *freq;

    /* per-sequence state: offsets in floats into the model's state (recurrent), device pointers of the latent cache */
    long long conv_state, rec_state;
    void *cache_c, *cache_kr;
} StackLayer;

typedef struct {
    int width, vocab, n_layers;
    float eps, embed_scale;
    StackLayer *layers;
} StackConfig;

/* 0 on success; otherwise an error is recorded and nothing is kept */
int ckb_stack_config_read(const char *path, StackConfig *out);
void ckb_stack_config_free(StackConfig *c);

#endif
