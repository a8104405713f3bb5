/* The layer-stack model family, inside: the model, the buffers of a pass, and what its three files share (model_stack_weights.c,
 * model_stack_mixers.c, model_stack.c). */
#ifndef CKB200_MODEL_STACK_H
#define CKB200_MODEL_STACK_H

#include <stddef.h>
#include <stdint.h>

#include "layer_stack.h"
#include "model_internal.h"
#include "safetensors.h"

/* a tensor's place inside a stacked matrix, and a vector's in the arena */
typedef struct { LinMat *mat; char name[64]; int rows, cols, row0, col0, half; } MatPart;       /* half: 0 gate, 1 up rows of SwiGLU blocks, -1 plain */
enum { VEC_ONE = 0, VEC_NOISE };
typedef struct { float **dst; char name[64]; int n, space, init; const float *host; } VecPart;  /* space: floats it takes */

/* buffers of a pass of up to `rows` rows */
typedef struct {
    int rows, splits;
    float *x, *x2;          /* residual rows; output norm: the two take turns */
    float *d;               /* output norm: a sublayer's output */
    float *z, *y, *g, *o, *qa, *part, *ss;
    void *h, *mf, *lr, *q16;
} PassBuf;

typedef struct {
    struct CKB200Model;     /* shared fields (model_internal.h) */
    StackConfig s;
    int f32;
    int portion;            /* most tokens per sequence of one pass */
    int lead;               /* rows at the start of sequences that keep fp32-like activations */
    LinMat embed, head;
    float *final_norm;
    uint8_t *arena;
    size_t arena_bytes;
    float *state;
    size_t state_floats;
    uint8_t *cache;
    size_t cache_bytes;
    /* the decode step's own buffers (its graph keeps the pointers), those of prompt passes, and of passes with so few rows that their
     * activations are fp32: a buffer only ever holds one activation type, so the zero-weighted pads of its rows stay finite */
    PassBuf dec, pre, few;
    int ld_x, ld_h, ld_z, ld_mf, ld_lr, ld_y, ld_g, ld_o, qa_row, part_row, ss_row, q16_row;
    uint8_t *expand;
    size_t expand_bytes;
    int32_t *ids, *want;    /* of prompt passes */
    int ids_cap;
    float *want_logits;
    MatPart *mats;
    VecPart *vecs;
    int n_mats, n_vecs;
    float *probe;           /* host: residual rows after every layer of the next prompt passes */
    int probe_rows, probe_at;
} StackModel;

/* T tokens of each of B sequences, row t * B + b */
typedef struct {
    int T, B, R, act;       /* act: activation type (linear.h) */
    const PassBuf *b;
    void *st;
    float *x, *other;       /* residual rows, and the buffer that takes them next (output norm) */
    const float *join;      /* output norm: norm weights of the output in b->d that has not joined x yet; NULL: none */
} Pass;

#define STACK_LATENT_ROWS 64        /* rows of a pass that go through absorbed latent attention together */
#define STACK_LOGIT_ROWS 128
#define STACK_MAX_SPLITS 64

static inline int pad8(int v) { return (v + 7) / 8 * 8; }
static inline int pad32(int v) { return (v + 31) / 32 * 32; }
static inline int pad64(int v) { return (v + 63) / 64 * 64; }
static inline size_t up256(size_t v) { return (v + 255) / 256 * 256; }
static inline int max2(int a, int b) { return a > b ? a : b; }
static inline void *act_at(const Pass *p, void *base, size_t col) { return (uint8_t *)base + col * (p->act == ACT_F32 ? 4 : 2); }
static inline void seg_from(LinSegs *sg, int x0, int row0, int count, int kind, void *dst, int ld)
{
    LinSeg *s = &sg->s[sg->n++];
    s->x0 = x0;
    s->row0 = row0;
    s->count = count;
    s->kind = kind;
    s->ld = ld;
    s->dst = dst;
}
static inline void seg_add(LinSegs *sg, int row0, int count, int kind, void *dst, int ld) { seg_from(sg, 0, row0, count, kind, dst, ld); }

/* model_stack_weights.c */
int ckb_stack_ranks_from_tensors(StackModel *m, const CkbSafetensors *st);
int ckb_stack_place_weights(StackModel *m, const CkbSafetensors *st, unsigned long long seed);     /* st NULL: random */
size_t ckb_stack_weight_elements(const StackModel *m);

/* model_stack_mixers.c */
int ckb_stack_plan_state(StackModel *m);
int ckb_stack_latent_splits(const StackModel *m, const StackMixer *x, int rows);
int ckb_stack_product(const LinMat *w, const void *x, int ldx, int rows, const LinSegs *sg, void *st);   /* x in the pass's activation type */
void ckb_stack_in_segments(const StackModel *m, const StackLayer *l, const Pass *p, LinSegs *sg);
/* From the projections (b->z, b->lr) to the input of the output projection (b->mf).  *scale_rest: set to the mixer whose columns still
 * need the RMS factor of b->ss, NULL when nothing is left to do */
int ckb_stack_mix(StackModel *m, StackLayer *l, const Pass *p, const StackMixer **scale_rest);

#endif
