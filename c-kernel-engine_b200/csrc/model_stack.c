/* The family of layer-stack decoders: a folder with config.json (layer_stack_config.c) and a bfloat16 model.safetensors, or
 * "synthetic:<path of a config.json>[:seed]" with random weights of those sizes.
 *
 * A layer is x += mixer(h) + ff(h), h = norm(x).  Everything that reads h is one stacked matrix (`in`: the mixer's projections, then the
 * feed-forward's gate and up rows with SwiGLU in the epilogue) and everything that is added to x is another (`out`: output projection
 * and down projection side by side over [mixer output | ff output], added to the residual in the epilogue), so a layer is two products
 * around the mixer's own steps (mixers.h).  The residual, norms, angles, scores, gates and recurrent state are fp32; the inputs of the
 * products are bfloat16 when there are many rows, fp32 when there are few or the model runs in 32-bit (tune key model_f32 at open).
 *
 * State of a sequence: recurrent states and convolution tails (fp32), and for latent attention one latent and one rotated key part per
 * position.  A pass carries T tokens of each of the `batch` sequences; row t * batch + b. */
#include <cuda_runtime_api.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>
#include <sys/stat.h>

#include "../../include/ckb200.h"
#include "launch.h"
#include "layer_stack.h"
#include "mixers.h"
#include "model_internal.h"
#include "runtime.h"
#include "safetensors.h"

#define STACK_LATENT_ROWS 64        /* rows of a pass that go through absorbed latent attention together */
#define STACK_LOGIT_ROWS 128
#define STACK_MAX_SPLITS 64

typedef struct { LinMat *mat; char name[64]; int rows, cols, row0, col0, half; } MatPart;       /* half: 0 gate, 1 up rows of SwiGLU blocks, -1 plain */
enum { VEC_ONE = 0, VEC_NOISE };
typedef struct { float **dst; char name[64]; int n, init; const float *host; } VecPart;

/* buffers of a pass of up to `rows` rows */
typedef struct {
    int rows, splits;
    float *x, *z, *y, *g, *o, *qa, *part;
    void *h, *mf, *lr;
} PassBuf;

typedef struct {
    struct CKB200Model;     /* shared fields (model_internal.h) */
    StackConfig s;
    int f32;
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
    int ld_x, ld_h, ld_z, ld_mf, ld_lr, ld_y, ld_g, ld_o, qa_row, part_row;
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

static int pad32(int v) { return (v + 31) / 32 * 32; }
static int pad64(int v) { return (v + 63) / 64 * 64; }
static size_t up256(size_t v) { return (v + 255) / 256 * 256; }
static int max2(int a, int b) { return a > b ? a : b; }

/* ------------------------------------------------------------------ placing the weights */

static MatPart *mat_part(StackModel *m, LinMat *mat, int rows, int cols, int row0, int col0, int half)
{
    MatPart *grown = (MatPart *)realloc(m->mats, (size_t)(m->n_mats + 1) * sizeof(MatPart));
    if (!grown) return NULL;
    m->mats = grown;
    MatPart *p = &m->mats[m->n_mats++];
    memset(p, 0, sizeof *p);
    p->mat = mat;
    p->rows = rows;
    p->cols = cols;
    p->row0 = row0;
    p->col0 = col0;
    p->half = half;
    return p;
}

/* a tensor's rows appended to a stacked matrix; returns their first row */
static int stack_rows(StackModel *m, LinMat *mat, int layer, const char *name, int rows, int cols)
{
    const int row0 = mat->rows;
    MatPart *p = mat_part(m, mat, rows, cols, row0, 0, -1);
    if (!p) return row0;
    if (layer >= 0) snprintf(p->name, sizeof p->name, "l%d.%s", layer, name);
    else snprintf(p->name, sizeof p->name, "%s", name);
    mat->rows += pad32(rows);
    mat->cols = max2(mat->cols, pad64(cols));
    return row0;
}

static void vec_part(StackModel *m, float **dst, int layer, const char *name, int n, int init, const float *host)
{
    VecPart *grown = (VecPart *)realloc(m->vecs, (size_t)(m->n_vecs + 1) * sizeof(VecPart));
    if (!grown) return;
    m->vecs = grown;
    VecPart *p = &m->vecs[m->n_vecs++];
    memset(p, 0, sizeof *p);
    p->dst = dst;
    p->n = n;
    p->init = init;
    p->host = host;
    if (layer >= 0) snprintf(p->name, sizeof p->name, "l%d.%s", layer, name);
    else snprintf(p->name, sizeof p->name, "%s", name);
}

static void plan_layer(StackModel *m, int i)
{
    StackLayer *l = &m->s.layers[i];
    const int D = m->s.width, H = l->heads, G = l->kv_heads, ov = H * l->vdim;
    vec_part(m, &l->norm1, i, "norm1", D, VEC_ONE, NULL);
    if (l->type == STACK_RETENTION) {
        l->row_q = stack_rows(m, &l->in, i, "mix.q", H * l->dim, D);
        l->row_k = stack_rows(m, &l->in, i, "mix.k", H * l->dim, D);
        l->row_v = stack_rows(m, &l->in, i, "mix.v", ov, D);
        l->row_g = stack_rows(m, &l->in, i, "mix.g", ov, D);
    } else if (l->type == STACK_LATENT_ATTENTION) {
        l->row_dq = stack_rows(m, &l->in, i, "mix.dq", l->q_rank, D);
        l->row_dkv = stack_rows(m, &l->in, i, "mix.dkv", l->kv_rank + l->rot_dim, D);
        stack_rows(m, &l->uq, i, "mix.uq", H * (l->dim + l->rot_dim), l->q_rank);
        stack_rows(m, &l->ukv, i, "mix.uk", H * l->dim, l->kv_rank);
        l->row_uv = stack_rows(m, &l->ukv, i, "mix.uv", ov, l->kv_rank);
        vec_part(m, &l->q_norm, i, "mix.dq.norm", l->q_rank, VEC_ONE, NULL);
        vec_part(m, &l->kv_norm, i, "mix.dkv.norm", l->kv_rank, VEC_ONE, NULL);
    } else {
        l->row_q = stack_rows(m, &l->in, i, "mix.q", G * l->dim, D);
        l->row_k = stack_rows(m, &l->in, i, "mix.k", G * l->dim, D);
        l->row_v = stack_rows(m, &l->in, i, "mix.v", ov, D);
        l->row_b = stack_rows(m, &l->in, i, "mix.b", H, D);
        l->row_a1 = stack_rows(m, &l->in, i, "mix.a1", l->a_rank, D);
        l->row_g1 = stack_rows(m, &l->in, i, "mix.g1", l->g_rank, D);
        stack_rows(m, &l->a2, i, "mix.a2", H * l->dim, l->a_rank);
        stack_rows(m, &l->g2, i, "mix.g2", ov, l->g_rank);
        vec_part(m, &l->a_log, i, "mix.A_log", H, VEC_NOISE, NULL);
        vec_part(m, &l->dt_bias, i, "mix.dt_bias", H * l->dim, VEC_NOISE, NULL);
        vec_part(m, &l->head_norm, i, "mix.norm", l->vdim, VEC_ONE, NULL);
        /* the three convolutions' filters are one table over all channels: their parts follow one another */
        vec_part(m, &l->conv_w, i, "mix.q.conv", G * l->dim * l->taps, VEC_NOISE, NULL);
        vec_part(m, NULL, i, "mix.k.conv", G * l->dim * l->taps, VEC_NOISE, NULL);
        vec_part(m, NULL, i, "mix.v.conv", ov * l->taps, VEC_NOISE, NULL);
    }
    l->z_width = l->in.rows;
    l->row_ff = l->in.rows;
    stack_rows(m, &l->out, i, "mix.o", D, ov);
    l->col_ff = l->out.cols;
    if (l->ff) {
        for (int half = 0; half < 2; ++half) {
            MatPart *p = mat_part(m, &l->in, l->ff, D, l->row_ff, 0, half);
            if (p) snprintf(p->name, sizeof p->name, "l%d.mlp.%s", i, half ? "up" : "gate");
        }
        l->in.rows += (l->ff + 15) / 16 * 32;
        MatPart *p = mat_part(m, &l->out, D, l->ff, 0, l->col_ff, -1);
        if (p) snprintf(p->name, sizeof p->name, "l%d.mlp.down", i);
        l->out.cols += pad64(l->ff);
    }
}

/* every matrix of the model, in arena order */
static int each_mat(StackModel *m, int k, LinMat **out)
{
    if (k == 0) { *out = &m->embed; return 1; }
    if (k == 1) { *out = &m->head; return 1; }
    k -= 2;
    if (k >= 6 * m->s.n_layers) return 0;
    StackLayer *l = &m->s.layers[k / 6];
    LinMat *list[6] = { &l->in, &l->out, &l->uq, &l->ukv, &l->a2, &l->g2 };
    *out = list[k % 6];
    return 1;
}

static int upload_mat(StackModel *m, const MatPart *p, const CkbSafetensors *st, unsigned long long seed)
{
    uint16_t *base = (uint16_t *)(uintptr_t)p->mat->w + (size_t)p->row0 * p->mat->cols + p->col0;
    const size_t pitch = (size_t)p->mat->cols * 2, width = (size_t)p->cols * 2;
    if (!st) {
        const float scale = p->mat == &m->embed ? 1.0f / m->s.embed_scale : 0.5f / __builtin_sqrtf((float)p->cols);
        return ckb_launch_fill_bf16(base, p->mat->cols, p->rows, p->cols, p->half, scale, seed, NULL);
    }
    CkbStTensor t;
    if (!ckb_st_find(st, p->name, &t)) return ckb_fail(CKB_ERR_STATE, "model: no tensor '%s'", p->name);
    if (strcmp(t.dtype, "BF16") || t.ndim != 2 || t.shape[0] != p->rows || t.shape[1] != p->cols || t.bytes != (size_t)p->rows * width)
        return ckb_fail(CKB_ERR_SHAPE, "model: tensor '%s' is not bfloat16 [%d, %d]", p->name, p->rows, p->cols);
    if (p->half < 0) return ckb_check_cuda((int)cudaMemcpy2D(base, pitch, t.data, width, width, (size_t)p->rows, cudaMemcpyHostToDevice), "upload matrix");
    for (int r = 0; r < p->rows; r += 16) {
        const size_t n = (size_t)(p->rows - r < 16 ? p->rows - r : 16);
        if (ckb_check_cuda((int)cudaMemcpy2D(base + ((size_t)r * 2 + 16 * p->half) * p->mat->cols, pitch, (const uint8_t *)t.data + (size_t)r * width, width, width, n,
                                             cudaMemcpyHostToDevice), "upload gate/up rows")) return CKB_ERR_CUDA;
    }
    return 0;
}

static int upload_vec(const VecPart *p, float *dev, const CkbSafetensors *st, unsigned long long seed)
{
    float *tmp = (float *)malloc((size_t)p->n * sizeof(float));
    if (!tmp) return ckb_fail(CKB_ERR_STATE, "model: out of memory");
    int rc = 0;
    if (p->host) {
        memcpy(tmp, p->host, (size_t)p->n * sizeof(float));
    } else if (!st) {
        unsigned long long r = seed * 6364136223846793005ull + 1442695040888963407ull;
        for (int i = 0; i < p->n; ++i) {
            r = r * 6364136223846793005ull + 1442695040888963407ull;
            const float u = (float)(r >> 40) / 16777216.0f - 0.5f;
            tmp[i] = p->init == VEC_ONE ? 1.0f + 0.2f * u : u;
        }
    } else {
        CkbStTensor t;
        if (!ckb_st_find(st, p->name, &t)) rc = ckb_fail(CKB_ERR_STATE, "model: no tensor '%s'", p->name);
        else if (strcmp(t.dtype, "BF16") || t.bytes != (size_t)p->n * 2) rc = ckb_fail(CKB_ERR_SHAPE, "model: tensor '%s' is not bfloat16 with %d elements", p->name, p->n);
        else
            for (int i = 0; i < p->n; ++i) {
                const uint32_t bits = (uint32_t)((const uint16_t *)t.data)[i] << 16;
                memcpy(&tmp[i], &bits, 4);
            }
    }
    if (!rc) rc = ckb_check_cuda((int)cudaMemcpy(dev, tmp, (size_t)p->n * sizeof(float), cudaMemcpyHostToDevice), "upload vector");
    free(tmp);
    return rc;
}

static int place_weights(StackModel *m, const CkbSafetensors *st, unsigned long long seed)
{
    size_t cur = 0;
    LinMat *mat;
    for (int k = 0; each_mat(m, k, &mat); ++k)
        if (mat->rows) { mat->w = (void *)(uintptr_t)cur; cur = up256(cur + (size_t)mat->rows * mat->cols * 2); }
    size_t *off = (size_t *)malloc((size_t)m->n_vecs * sizeof(size_t));
    if (!off) return ckb_fail(CKB_ERR_STATE, "model: out of memory");
    for (int i = 0; i < m->n_vecs; ++i) {
        if (m->vecs[i].dst) cur = up256(cur);
        off[i] = cur;
        cur += (size_t)m->vecs[i].n * sizeof(float);
    }
    m->arena_bytes = cur + 256;
    int rc = ckb_check_cuda((int)cudaMalloc((void **)&m->arena, m->arena_bytes), "cudaMalloc(weights)");
    if (!rc) rc = ckb_check_cuda((int)cudaMemset(m->arena, 0, m->arena_bytes), "zero weights");
    for (int k = 0; !rc && each_mat(m, k, &mat); ++k)
        if (mat->rows) { mat->w = m->arena + (uintptr_t)mat->w; rc = ckb_linear_encode(mat); }
    if (!rc) rc = ckb_check_cuda((int)cudaDeviceSynchronize(), "zero weights");
    for (int i = 0; !rc && i < m->n_mats; ++i) rc = upload_mat(m, &m->mats[i], st, seed * 7919 + (unsigned long long)i);
    for (int i = 0; !rc && i < m->n_vecs; ++i) {
        float *dev = (float *)(m->arena + off[i]);
        if (m->vecs[i].dst) *m->vecs[i].dst = dev;
        rc = upload_vec(&m->vecs[i], dev, st, seed * 104729 + (unsigned long long)i);
    }
    free(off);
    return rc;
}

/* ------------------------------------------------------------------ buffers */

static int latent_splits(const StackModel *m, const StackLayer *l, int rows)
{
    const int groups = rows * ((l->heads + 15) / 16);
    int s = 2 * ckb_sm_count() / groups, most = (m->c.max_seq_len + 63) / 64;
    if (s > most) s = most;
    if (s > STACK_MAX_SPLITS) s = STACK_MAX_SPLITS;
    return s < 1 ? 1 : s;
}

static void pass_free(PassBuf *p)
{
    void *ptrs[] = { p->x, p->z, p->y, p->g, p->o, p->qa, p->part, p->h, p->mf, p->lr };
    for (size_t i = 0; i < sizeof ptrs / sizeof ptrs[0]; ++i) if (ptrs[i]) cudaFree(ptrs[i]);
    memset(p, 0, sizeof *p);
}

static int pass_alloc(StackModel *m, PassBuf *p, int rows)
{
    if (rows <= p->rows) return 0;
    cudaStream_t st = ckb_stream(NULL);
    cudaStreamSynchronize(st);
    pass_free(p);
    const size_t R = (size_t)rows, lat = R < STACK_LATENT_ROWS ? R : STACK_LATENT_ROWS;
    p->splits = 1;
    for (int i = 0; i < m->s.n_layers; ++i)
        if (m->s.layers[i].type == STACK_LATENT_ATTENTION) p->splits = max2(p->splits, latent_splits(m, &m->s.layers[i], (int)lat));
    struct { void **p; size_t bytes; } need[] = {
        { (void **)&p->x, R * m->ld_x * 4 }, { (void **)&p->h, R * m->ld_h * 4 }, { (void **)&p->z, R * m->ld_z * 4 }, { (void **)&p->mf, R * m->ld_mf * 4 },
        { (void **)&p->lr, R * m->ld_lr * 4 }, { (void **)&p->y, R * m->ld_y * 4 }, { (void **)&p->g, R * m->ld_g * 4 }, { (void **)&p->o, R * m->ld_o * 4 },
        { (void **)&p->qa, lat * m->qa_row * 4 }, { (void **)&p->part, lat * p->splits * m->part_row * 4 },
    };
    for (size_t i = 0; i < sizeof need / sizeof need[0]; ++i) {
        if (!need[i].bytes) continue;
        if (ckb_check_cuda((int)cudaMalloc(need[i].p, need[i].bytes + 256), "cudaMalloc(pass)") ||
            ckb_check_cuda((int)cudaMemsetAsync(*need[i].p, 0, need[i].bytes + 256, st), "zero pass buffers")) {       /* pads of rows stay finite */
            pass_free(p);
            return CKB_ERR_CUDA;
        }
    }
    p->rows = rows;
    return 0;
}

static int plan_state(StackModel *m)
{
    const size_t B = (size_t)m->c.batch, eb = m->f32 ? 4 : 2;
    size_t fl = 0, cb = 0;
    m->ld_x = m->ld_h = pad64(m->s.width);
    for (int i = 0; i < m->s.n_layers; ++i) {
        StackLayer *l = &m->s.layers[i];
        const int H = l->heads, G = l->kv_heads, ov = pad32(H * l->vdim);
        m->ld_z = max2(m->ld_z, l->z_width);
        m->ld_mf = max2(m->ld_mf, l->out.cols);
        m->ld_o = max2(m->ld_o, ov);
        if (l->type == STACK_LATENT_ATTENTION) {
            m->ld_lr = max2(m->ld_lr, l->uq.cols);
            m->ld_y = max2(m->ld_y, l->uq.rows);
            m->qa_row = max2(m->qa_row, H * (pad64(l->kv_rank) + pad32(l->rot_dim)));
            m->part_row = max2(m->part_row, H * (l->kv_rank + 2));
            l->cache_c = (void *)(uintptr_t)cb;
            cb = up256(cb + B * m->c.max_seq_len * pad64(l->kv_rank) * eb);
            l->cache_kr = (void *)(uintptr_t)cb;
            cb = up256(cb + B * m->c.max_seq_len * pad32(l->rot_dim) * eb);
            continue;
        }
        if (l->type == STACK_CHANNEL_DELTA) {
            const size_t channels = 2 * (size_t)G * l->dim + (size_t)H * l->vdim;
            m->ld_lr = max2(m->ld_lr, l->a2.cols + l->g2.cols);
            m->ld_y = max2(m->ld_y, 2 * pad32(G * l->dim) + ov);
            m->ld_g = max2(m->ld_g, l->a2.rows + l->g2.rows);
            l->conv_state = (long long)fl;
            fl += (B * l->taps * channels + 63) / 64 * 64;
        }
        l->rec_state = (long long)fl;
        fl += B * H * l->vdim * ckb_recur_dp(l->dim);
    }
    m->state_floats = fl;
    m->cache_bytes = cb;
    if (fl && ckb_check_cuda((int)cudaMalloc((void **)&m->state, fl * 4), "cudaMalloc(state)")) return CKB_ERR_CUDA;
    if (fl && ckb_check_cuda((int)cudaMemset(m->state, 0, fl * 4), "zero state")) return CKB_ERR_CUDA;
    if (cb && ckb_check_cuda((int)cudaMalloc((void **)&m->cache, cb), "cudaMalloc(cache)")) return CKB_ERR_CUDA;
    if (cb && ckb_check_cuda((int)cudaMemset(m->cache, 0, cb), "zero cache")) return CKB_ERR_CUDA;
    for (int i = 0; i < m->s.n_layers; ++i) {
        StackLayer *l = &m->s.layers[i];
        if (l->type != STACK_LATENT_ATTENTION) continue;
        l->cache_c = m->cache + (uintptr_t)l->cache_c;
        l->cache_kr = m->cache + (uintptr_t)l->cache_kr;
    }
    return pass_alloc(m, &m->dec, m->c.batch);
}

/* ------------------------------------------------------------------ a pass over T tokens of each sequence */

typedef struct { int T, B, R, act_f32; const PassBuf *b; void *st; } Pass;

/* y = W x for the rows of a pass; x in the pass's activation type */
static int product(const LinMat *w, const void *x, int ldx, int rows, const LinSegs *sg, void *st)
{
    if (rows <= LIN_GEMV_MAX_TOKENS) return ckb_launch_linear_gemv(w, (const float *)x, ldx, rows, NULL, 0, 0.f, sg, st);
    return sg->act_f32 ? ckb_launch_linear_f32(w, (const float *)x, ldx, rows, sg, st) : ckb_launch_linear_tc(w, x, ldx, rows, sg, st);
}

static void seg_add(LinSegs *sg, int row0, int count, int kind, void *dst, int ld)
{
    LinSeg *s = &sg->s[sg->n++];
    s->row0 = row0;
    s->count = count;
    s->kind = kind;
    s->ld = ld;
    s->dst = dst;
}

static void *act_at(const Pass *p, void *base, int col) { return (uint8_t *)base + (size_t)col * (p->act_f32 ? 4 : 2); }

/* segments of the mixer's projections inside `in` */
static void in_segments(const StackModel *m, const StackLayer *l, const Pass *p, LinSegs *sg)
{
    float *z = p->b->z;
    const int ld = m->ld_z, H = l->heads, ov = H * l->vdim;
    if (l->type == STACK_RETENTION) {
        seg_add(sg, l->row_q, H * l->dim, LIN_F32, z + l->row_q, ld);
        seg_add(sg, l->row_k, H * l->dim, LIN_F32, z + l->row_k, ld);
        seg_add(sg, l->row_v, ov, LIN_F32, z + l->row_v, ld);
        seg_add(sg, l->row_g, ov, LIN_F32, z + l->row_g, ld);
    } else if (l->type == STACK_LATENT_ATTENTION) {
        seg_add(sg, l->row_dq, l->q_rank, LIN_F32, z + l->row_dq, ld);
        seg_add(sg, l->row_dkv, l->kv_rank + l->rot_dim, LIN_F32, z + l->row_dkv, ld);
    } else {
        seg_add(sg, l->row_q, l->kv_heads * l->dim, LIN_F32, z + l->row_q, ld);
        seg_add(sg, l->row_k, l->kv_heads * l->dim, LIN_F32, z + l->row_k, ld);
        seg_add(sg, l->row_v, ov, LIN_F32, z + l->row_v, ld);
        seg_add(sg, l->row_b, H, LIN_F32, z + l->row_b, ld);
        seg_add(sg, l->row_a1, l->a_rank, LIN_ACT, p->b->lr, m->ld_lr);
        seg_add(sg, l->row_g1, l->g_rank, LIN_ACT, act_at(p, p->b->lr, l->a2.cols), m->ld_lr);
    }
}

static LatentCache latent_cache(const StackModel *m, const StackLayer *l)
{
    LatentCache lc = { .H = l->heads, .dim = l->dim, .rot = l->rot_dim, .vdim = l->vdim, .rank = l->kv_rank, .rank_ld = pad64(l->kv_rank), .rot_ld = pad32(l->rot_dim),
                             .cap = m->c.max_seq_len, .cache_f32 = m->f32, .c = l->cache_c, .kr = l->cache_kr, .freq = l->freq, .scale = l->scale };
    lc.q_split = ckb_latent_q_split(&lc);
    return lc;
}

static int retention_rows(StackModel *m, StackLayer *l, const Pass *p)
{
    const PassBuf *b = p->b;
    float *z = b->z;
    const RotateRows rot[2] = {
        { .x = z + l->row_q, .ld = m->ld_z, .heads = l->heads, .head_stride = l->dim, .n = l->dim, .dims = l->rot_dims, .freq = l->freq, .mul = 1.0f },
        { .x = z + l->row_k, .ld = m->ld_z, .heads = l->heads, .head_stride = l->dim, .n = l->dim, .dims = l->rot_dims, .freq = l->freq, .mul = 1.0f / __builtin_sqrtf((float)l->dim) },
    };
    const RecurRows rec = { .q = z + l->row_q, .k = z + l->row_k, .v = z + l->row_v, .ldq = m->ld_z, .ldk = m->ld_z, .ldv = m->ld_z, .decay = l->decay, .G = l->heads,
                            .H = l->heads, .d = l->dim, .dv = l->vdim, .state = m->state + l->rec_state, .o = b->o, .ldo = m->ld_o };
    int rc = ckb_launch_rotate_rows(rot, 2, p->R, p->B, m->pos_dev, p->st);
    if (!rc) rc = ckb_launch_recur_rows(&rec, p->T, p->B, p->st);
    if (!rc) rc = ckb_launch_head_norm_gate(b->o, m->ld_o, NULL, z + l->row_g, m->ld_z, GATE_SILU, m->s.eps, l->heads, l->vdim, b->mf, l->out.cols, p->act_f32, p->R, p->st);
    return rc;
}

/* one token per sequence: the mixer's own steps in one launch */
static int recurrent_step(StackModel *m, StackLayer *l, const Pass *p)
{
    const PassBuf *b = p->b;
    float *z = b->z;
    const int ld = m->ld_z;
    const RecurStep s = {
        .r = { .q = z + l->row_q, .k = z + l->row_k, .v = z + l->row_v, .ldq = ld, .ldk = ld, .ldv = ld, .decay = l->decay, .G = l->kv_heads, .H = l->heads, .d = l->dim, .dv = l->vdim,
               .state = m->state + l->rec_state },
        .delta = l->type == STACK_CHANNEL_DELTA, .freq = l->freq, .rot_dims = l->rot_dims, .gate = z + l->row_g, .conv_w = l->conv_w, .conv_state = m->state + l->conv_state, .taps = l->taps,
        .beta = z + l->row_b, .a_low = (const float *)b->lr, .g_low = (const float *)b->lr + l->a2.cols, .a2 = l->a2.w, .g2 = l->g2.w, .ld_a2 = l->a2.cols, .ld_g2 = l->g2.cols,
        .a_log = l->a_log, .dt_bias = l->dt_bias, .head_norm = l->head_norm, .ldz = ld, .ld_low = m->ld_lr, .eps = m->s.eps, .dst = b->mf, .ldd = l->out.cols, .act_f32 = p->act_f32,
    };
    return ckb_launch_recur_step(&s, p->B, m->pos_dev, p->st);
}

static int step_takes(const StackLayer *l, const Pass *p)
{
    if (p->T != 1 || !p->act_f32 || !ckb_tune_get("stack_fused_step", 1)) return 0;
    return l->type == STACK_LATENT_ATTENTION || (ckb_recur_step_takes(l->dim, l->vdim) && l->a2.cols + l->g2.cols <= 8192);
}

static int channel_delta_rows(StackModel *m, StackLayer *l, const Pass *p)
{
    const PassBuf *b = p->b;
    float *z = b->z, *yq = b->y, *yk = yq + pad32(l->kv_heads * l->dim), *yv = yk + pad32(l->kv_heads * l->dim), *gate = b->g + l->a2.rows;
    LinSegs sa = { .act_f32 = p->act_f32 }, sgate = sa;
    seg_add(&sa, 0, l->heads * l->dim, LIN_F32, b->g, m->ld_g);
    seg_add(&sgate, 0, l->heads * l->vdim, LIN_F32, gate, m->ld_g);
    const ConvRows cv = { .q = z + l->row_q, .k = z + l->row_k, .v = z + l->row_v, .ld = m->ld_z, .w = l->conv_w, .state = m->state + l->conv_state, .oq = yq, .ok = yk, .ov = yv,
                          .ldo = m->ld_y, .G = l->kv_heads, .H = l->heads, .d = l->dim, .dv = l->vdim, .taps = l->taps };
    const RecurRows rec = { .q = yq, .k = yk, .v = yv, .g = b->g, .beta = z + l->row_b, .ldq = m->ld_y, .ldk = m->ld_y, .ldv = m->ld_y, .ldg = m->ld_g, .ldb = m->ld_z,
                            .G = l->kv_heads, .H = l->heads, .d = l->dim, .dv = l->vdim, .state = m->state + l->rec_state, .o = b->o, .ldo = m->ld_o };
    int rc = product(&l->a2, b->lr, m->ld_lr, p->R, &sa, p->st);
    if (!rc) rc = product(&l->g2, act_at(p, b->lr, l->a2.cols), m->ld_lr, p->R, &sgate, p->st);
    if (!rc) rc = ckb_launch_conv_rows(&cv, p->T, p->B, m->pos_dev, p->st);
    if (!rc) rc = ckb_launch_delta_gates(b->g, m->ld_g, l->a_log, l->dt_bias, l->heads, l->dim, z + l->row_b, m->ld_z, p->R, p->st);
    if (!rc) rc = ckb_launch_recur_rows(&rec, p->T, p->B, p->st);
    if (!rc) rc = ckb_launch_head_norm_gate(b->o, m->ld_o, l->head_norm, gate, m->ld_g, GATE_SIGMOID, m->s.eps, l->heads, l->vdim, b->mf, l->out.cols, p->act_f32, p->R, p->st);
    return rc;
}

/* keys and values of a whole sequence for the expanded form of latent attention: grown on demand, shared by the layers */
static int expand_alloc(StackModel *m, size_t bytes)
{
    if (bytes <= m->expand_bytes) return 0;
    cudaStreamSynchronize(ckb_stream(NULL));
    if (m->expand) cudaFree(m->expand);
    m->expand = NULL;
    m->expand_bytes = 0;
    bytes += bytes / 4;
    if (ckb_check_cuda((int)cudaMalloc((void **)&m->expand, bytes), "cudaMalloc(expanded keys)")) return CKB_ERR_CUDA;
    m->expand_bytes = bytes;
    return 0;
}

static int latent_expanded(StackModel *m, StackLayer *l, const LatentCache *lc, const Pass *p)
{
    const PassBuf *b = p->b;
    const size_t keys = (size_t)m->host_pos + p->T, kw = (size_t)l->heads * l->dim, vw = (size_t)l->heads * l->vdim, qw = (size_t)l->heads * (l->dim + l->rot_dim);
    const size_t kb = up256(keys * kw * 2), vb = up256(keys * vw * 2);
    int rc = expand_alloc(m, kb + vb + up256(p->R * qw * 2));
    if (rc) return rc;
    uint8_t *k = m->expand, *v = k + kb, *q = v + vb;
    rc = ckb_launch_latent_query(lc, b->y, m->ld_y, q, p->R, p->B, m->pos_dev, p->st);
    for (int i = 0; !rc && i < p->B; ++i) {
        LinSegs sg = { .act_f32 = 0 };
        seg_add(&sg, 0, (int)kw, LIN_ACT, k, (int)kw);
        seg_add(&sg, l->row_uv, (int)vw, LIN_ACT, v, (int)vw);
        rc = ckb_launch_linear_tc(&l->ukv, (const uint16_t *)lc->c + (size_t)i * lc->cap * lc->rank_ld, lc->rank_ld, (int)keys, &sg, p->st);
        if (!rc) rc = ckb_launch_latent_prefill(lc, q, k, v, b->mf, l->out.cols, p->T, p->B, i, m->pos_dev, p->st);
    }
    return rc;
}

static int latent_rows(StackModel *m, StackLayer *l, const Pass *p)
{
    const PassBuf *b = p->b;
    const LatentCache lc = latent_cache(m, l);
    LinSegs sq = { .act_f32 = p->act_f32 };
    seg_add(&sq, 0, l->heads * (l->dim + l->rot_dim), LIN_F32, b->y, m->ld_y);
    const uint16_t *uk = (const uint16_t *)l->ukv.w, *uv = uk + (size_t)l->row_uv * l->ukv.cols;
    int rc;
    if (p->R <= LIN_GEMV_MAX_TOKENS && step_takes(l, p)) {
        const int splits = max2(1, latent_splits(m, l, p->R) < b->splits ? latent_splits(m, l, p->R) : b->splits);
        rc = ckb_launch_linear_gemv(&l->uq, b->z + l->row_dq, m->ld_z, p->R, l->q_norm, l->q_rank, m->s.eps, &sq, p->st);
        if (!rc) rc = ckb_launch_latent_absorb_append(&lc, b->y, m->ld_y, uk, l->ukv.cols, b->qa, b->z + l->row_dkv, m->ld_z, l->kv_norm, m->s.eps, p->R, p->B, m->pos_dev, p->st);
        if (!rc) rc = ckb_launch_latent_attend(&lc, b->qa, b->part, splits, p->R, 0, p->B, m->pos_dev, p->st);
        return rc ? rc : ckb_launch_latent_output(&lc, b->part, splits, uv, l->ukv.cols, b->mf, l->out.cols, p->act_f32, p->R, 0, p->B, m->pos_dev, p->st);
    }
    rc = ckb_launch_rms_rows(b->z + l->row_dq, m->ld_z, NULL, p->R, l->q_rank, l->q_norm, m->s.eps, b->lr, m->ld_lr, l->uq.cols, p->act_f32, p->st);
    if (!rc) rc = product(&l->uq, b->lr, m->ld_lr, p->R, &sq, p->st);
    if (!rc) rc = ckb_launch_latent_append(&lc, b->z + l->row_dkv, m->ld_z, l->kv_norm, m->s.eps, p->R, p->B, m->pos_dev, p->st);
    if (!rc && !p->act_f32 && p->b == &m->pre && ckb_latent_prefill_takes(&lc)) return latent_expanded(m, l, &lc, p);
    for (int r0 = 0; !rc && r0 < p->R; r0 += STACK_LATENT_ROWS) {
        const int n = p->R - r0 < STACK_LATENT_ROWS ? p->R - r0 : STACK_LATENT_ROWS;
        const int splits = max2(1, latent_splits(m, l, n) < b->splits ? latent_splits(m, l, n) : b->splits);
        rc = ckb_launch_latent_absorb(&lc, b->y, m->ld_y, uk, l->ukv.cols, b->qa, n, r0, p->B, m->pos_dev, p->st);
        if (!rc) rc = ckb_launch_latent_attend(&lc, b->qa, b->part, splits, n, r0, p->B, m->pos_dev, p->st);
        if (!rc) rc = ckb_launch_latent_output(&lc, b->part, splits, uv, l->ukv.cols, act_at(p, b->mf, r0 * l->out.cols), l->out.cols, p->act_f32, n, r0, p->B, m->pos_dev, p->st);
    }
    return rc;
}

static int issue_rows(StackModel *m, const Pass *p, const int32_t *ids)
{
    const StackConfig *s = &m->s;
    const PassBuf *b = p->b;
    int rc = ckb_launch_embed_rows(ids, p->R, s->vocab, m->embed.w, m->embed.cols, s->width, s->embed_scale, b->x, m->ld_x, p->st);
    for (int i = 0; !rc && i < s->n_layers; ++i) {
        StackLayer *l = &s->layers[i];
        LinSegs in = { .act_f32 = p->act_f32 }, out = in;
        in_segments(m, l, p, &in);
        if (l->ff) seg_add(&in, l->row_ff, l->ff, LIN_SWIGLU, act_at(p, b->mf, l->col_ff), l->out.cols);
        seg_add(&out, 0, s->width, LIN_ADD, b->x, m->ld_x);
        if (p->R <= LIN_GEMV_MAX_TOKENS) {
            rc = ckb_launch_linear_gemv(&l->in, b->x, m->ld_x, p->R, l->norm1, s->width, s->eps, &in, p->st);
        } else {
            rc = ckb_launch_rms_rows(b->x, m->ld_x, NULL, p->R, s->width, l->norm1, s->eps, b->h, m->ld_h, m->ld_h, p->act_f32, p->st);
            if (!rc) rc = product(&l->in, b->h, m->ld_h, p->R, &in, p->st);
        }
        if (!rc && l->type != STACK_LATENT_ATTENTION && step_takes(l, p)) rc = recurrent_step(m, l, p);
        else if (!rc) rc = l->type == STACK_RETENTION ? retention_rows(m, l, p) : (l->type == STACK_LATENT_ATTENTION ? latent_rows(m, l, p) : channel_delta_rows(m, l, p));
        if (!rc) rc = product(&l->out, b->mf, l->out.cols, p->R, &out, p->st);
        if (!rc && m->probe && m->probe_at + p->R <= m->probe_rows)
            rc = ckb_check_cuda((int)cudaMemcpy2DAsync(m->probe + ((size_t)i * m->probe_rows + m->probe_at) * s->width, (size_t)s->width * 4, b->x, (size_t)m->ld_x * 4,
                                                       (size_t)s->width * 4, (size_t)p->R, cudaMemcpyDeviceToHost, (cudaStream_t)p->st), "residual probe");
    }
    if (m->probe && m->probe_at + p->R <= m->probe_rows) m->probe_at += p->R;
    return rc;
}

static int issue_logits(StackModel *m, const Pass *p, const int32_t *rows_dev, int n, float *logits)
{
    const PassBuf *b = p->b;
    LinSegs sg = { .act_f32 = m->f32 || n <= LIN_GEMV_MAX_TOKENS };
    seg_add(&sg, 0, m->s.vocab, LIN_F32, logits, m->s.vocab);
    if (!rows_dev && n <= LIN_GEMV_MAX_TOKENS) return ckb_launch_linear_gemv(&m->head, b->x, m->ld_x, n, m->final_norm, m->s.width, m->s.eps, &sg, p->st);
    const int rc = ckb_launch_rms_rows(b->x, m->ld_x, rows_dev, n, m->s.width, m->final_norm, m->s.eps, b->h, m->ld_h, m->ld_h, sg.act_f32, p->st);
    return rc ? rc : product(&m->head, b->h, m->ld_h, n, &sg, p->st);
}

static int stack_issue_step(CKB200Model *model, void *st)
{
    StackModel *m = (StackModel *)model;
    const int B = m->c.batch;
    const Pass p = { .T = 1, .B = B, .R = B, .act_f32 = m->f32 || B <= LIN_GEMV_MAX_TOKENS, .b = &m->dec, .st = st };
    int rc = issue_rows(m, &p, m->tokens_dev);
    if (!rc) rc = issue_logits(m, &p, NULL, B, m->logits);
    return rc ? rc : ckb_launch_advance_pos(m->pos_dev, 1, st);
}

static int stack_extend(CKB200Model *model, const int32_t *tokens, int count, const int32_t *want, int n_want, float *logits_host)
{
    StackModel *m = (StackModel *)model;
    const int B = m->c.batch, V = m->s.vocab;
    cudaStream_t st = ckb_stream(NULL);
    int portion = ckb_tune_get("stack_portion", 2048) / B;
    if (portion < 1) portion = 1;
    if (portion > count) portion = count;
    if (portion * B > LIN_GEMV_MAX_TOKENS && pass_alloc(m, &m->pre, portion * B)) return CKB_ERR_CUDA;
    if (pass_alloc(m, &m->few, LIN_GEMV_MAX_TOKENS)) return CKB_ERR_CUDA;
    if (m->ids_cap < portion * B) {
        if (m->ids) cudaFree(m->ids);
        if (m->want) cudaFree(m->want);
        m->ids = m->want = NULL;
        m->ids_cap = 0;
        if (ckb_check_cuda((int)cudaMalloc((void **)&m->ids, (size_t)portion * B * 4), "cudaMalloc(ids)") ||
            ckb_check_cuda((int)cudaMalloc((void **)&m->want, (size_t)portion * B * 4), "cudaMalloc(wanted rows)")) return CKB_ERR_CUDA;
        m->ids_cap = portion * B;
    }
    if (!m->want_logits && n_want && ckb_check_cuda((int)cudaMalloc((void **)&m->want_logits, (size_t)STACK_LOGIT_ROWS * V * 4), "cudaMalloc(logits)")) return CKB_ERR_CUDA;
    int32_t *rows = (int32_t *)malloc((size_t)portion * B * sizeof(int32_t));
    if (!rows) return ckb_fail(CKB_ERR_STATE, "model_extend: out of memory");
    int rc = 0, w = 0;
    for (int t0 = 0; !rc && t0 < count; t0 += portion) {
        const int T = count - t0 < portion ? count - t0 : portion, R = T * B;
        const Pass p = { .T = T, .B = B, .R = R, .act_f32 = m->f32 || R <= LIN_GEMV_MAX_TOKENS, .b = R <= LIN_GEMV_MAX_TOKENS ? &m->few : &m->pre, .st = st };
        rc = ckb_check_cuda((int)cudaMemcpyAsync(m->ids, tokens + (size_t)t0 * B, (size_t)R * 4, cudaMemcpyHostToDevice, st), "ids H2D");
        if (!rc) rc = issue_rows(m, &p, m->ids);
        int n = 0;
        for (; w < n_want && want[w] < t0 + T; ++w)
            for (int i = 0; i < B; ++i) rows[n++] = (want[w] - t0) * B + i;
        if (!rc && n) rc = ckb_check_cuda((int)cudaMemcpyAsync(m->want, rows, (size_t)n * 4, cudaMemcpyHostToDevice, st), "wanted rows H2D");
        for (int i = 0; !rc && i < n; i += STACK_LOGIT_ROWS) {
            const int k = n - i < STACK_LOGIT_ROWS ? n - i : STACK_LOGIT_ROWS;
            rc = issue_logits(m, &p, m->want + i, k, m->want_logits);
            if (!rc) rc = ckb_check_cuda((int)cudaMemcpyAsync(logits_host, m->want_logits, (size_t)k * V * 4, cudaMemcpyDeviceToHost, st), "logits D2H");
            logits_host += (size_t)k * V;
        }
        if (!rc) rc = ckb_launch_advance_pos(m->pos_dev, T, st);
        if (!rc) rc = ckb_sync_check(st, "model_extend");
        if (!rc) m->host_pos += T;
    }
    free(rows);
    return rc;
}

/* ------------------------------------------------------------------ opening */

static void stack_destroy(CKB200Model *model)
{
    StackModel *m = (StackModel *)model;
    pass_free(&m->dec);
    pass_free(&m->pre);
    pass_free(&m->few);
    void *ptrs[] = { m->arena, m->state, m->cache, m->expand, m->ids, m->want, m->want_logits };
    for (size_t i = 0; i < sizeof ptrs / sizeof ptrs[0]; ++i) if (ptrs[i]) cudaFree(ptrs[i]);
    ckb_stack_config_free(&m->s);
    free(m->mats);
    free(m->vecs);
}

static const char *synthetic_config(const char *spec, char *path, size_t cap, unsigned long long *seed)
{
    if (strncmp(spec, "synthetic:", 10)) return NULL;
    const char *end = strstr(spec + 10, ".json");
    if (!end || (size_t)(end + 5 - (spec + 10)) >= cap) return NULL;
    snprintf(path, cap, "%.*s", (int)(end + 5 - (spec + 10)), spec + 10);
    *seed = end[5] == ':' ? strtoull(end + 6, NULL, 10) : 1;
    return path;
}

static int stack_claims(const char *spec)
{
    char path[4096];
    unsigned long long seed;
    struct stat sb;
    if (synthetic_config(spec, path, sizeof path, &seed)) return 1;
    snprintf(path, sizeof path, "%s/config.json", spec);
    return stat(path, &sb) == 0;
}

/* low ranks that only the tensors tell */
static int ranks_from_tensors(StackModel *m, const CkbSafetensors *st)
{
    for (int i = 0; i < m->s.n_layers; ++i) {
        StackLayer *l = &m->s.layers[i];
        if (l->type != STACK_CHANNEL_DELTA) continue;
        if (st) {
            char name[64];
            CkbStTensor t;
            for (int k = 0; k < 2; ++k) {
                snprintf(name, sizeof name, "l%d.mix.%s", i, k ? "g1" : "a1");
                if (!ckb_st_find(st, name, &t) || t.ndim != 2 || t.shape[0] < 1 || t.shape[0] > 65536) return ckb_fail(CKB_ERR_STATE, "model: no tensor '%s'", name);
                *(k ? &l->g_rank : &l->a_rank) = (int)t.shape[0];
            }
        } else {
            if (l->a_rank <= 0) l->a_rank = l->dim;
            if (l->g_rank <= 0) l->g_rank = l->vdim;
        }
    }
    return 0;
}

static CKB200Model *stack_open(const char *spec, int batch)
{
    char cfg[4096], weights[4096];
    unsigned long long seed = 0;
    const int synth = synthetic_config(spec, cfg, sizeof cfg, &seed) != NULL;
    if (!synth) {
        snprintf(cfg, sizeof cfg, "%s/config.json", spec);
        snprintf(weights, sizeof weights, "%s/model.safetensors", spec);
    }
    StackConfig sc;
    if (ckb_stack_config_read(cfg, &sc)) return NULL;
    StackModel *m = (StackModel *)calloc(1, sizeof *m);
    CkbSafetensors *st = NULL;
    if (!m) { ckb_stack_config_free(&sc); return NULL; }
    m->family = &ckb_family_stack;
    m->s = sc;
    m->f32 = ckb_tune_get("model_f32", 0) != 0;
    m->c.embed_dim = sc.width;
    m->c.vocab_size = sc.vocab;
    m->c.num_layers = sc.n_layers;
    m->c.num_heads = m->c.num_kv_heads = sc.layers[0].heads;
    m->c.head_dim = sc.layers[0].dim;
    m->c.intermediate_size = sc.layers[0].ff;
    m->c.rms_eps = sc.eps;
    m->c.batch = batch > 0 ? batch : 1;
    m->c.tp_size = 1;
    m->c.max_seq_len = ckb_tune_get("model_max_seq", 4096);
    int rc = m->c.max_seq_len < 1 ? ckb_fail(CKB_ERR_SHAPE, "model_max_seq: %d", m->c.max_seq_len) : 0;
    if (!rc && !synth && !(st = ckb_st_open(weights))) rc = CKB_ERR_STATE;
    if (!rc) rc = ranks_from_tensors(m, st);
    float **freqs = (float **)calloc((size_t)sc.n_layers, sizeof(float *));
    if (!rc && !freqs) rc = ckb_fail(CKB_ERR_STATE, "model: out of memory");
    if (!rc) {
        stack_rows(m, &m->embed, -1, "embed", sc.vocab, sc.width);
        stack_rows(m, &m->head, -1, "head", sc.vocab, sc.width);
        vec_part(m, &m->final_norm, -1, "final.norm", sc.width, VEC_ONE, NULL);
        for (int i = 0; i < sc.n_layers && !rc; ++i) {
            StackLayer *l = &m->s.layers[i];
            plan_layer(m, i);
            if (l->decay_host) vec_part(m, &l->decay, i, "decay", l->heads, VEC_ONE, l->decay_host);
            if (l->rot_dims) {
                const int half = l->rot_dims / 2;
                freqs[i] = (float *)malloc((size_t)half * sizeof(float));
                if (!freqs[i]) { rc = ckb_fail(CKB_ERR_STATE, "model: out of memory"); break; }
                for (int k = 0; k < half; ++k) freqs[i][k] = (float)__builtin_pow(l->rot_base, -2.0 * k / l->rot_dims);
                vec_part(m, &l->freq, i, "freq", half, VEC_ONE, freqs[i]);
            }
        }
    }
    if (!rc && ckb_ensure_init()) rc = CKB_ERR_NO_DEVICE;
    if (!rc) rc = place_weights(m, st, seed);
    if (!rc) rc = ckb_model_init_shared((CKB200Model *)m);
    if (!rc) rc = plan_state(m);
    if (!rc) rc = ckb_check_cuda((int)cudaStreamSynchronize(ckb_stream(NULL)), "model init");
    for (int i = 0; freqs && i < sc.n_layers; ++i) free(freqs[i]);
    free(freqs);
    if (st) ckb_st_close(st);
    if (rc) {
        ckb200_model_free((CKB200Model *)m);
        return NULL;
    }
    return (CKB200Model *)m;
}

static int stack_clear_state(CKB200Model *model, void *st)
{
    StackModel *m = (StackModel *)model;
    m->probe_at = 0;
    return m->state ? ckb_check_cuda((int)cudaMemsetAsync(m->state, 0, m->state_floats * 4, (cudaStream_t)st), "clear state") : 0;
}

static int stack_can_set_pos(const CKB200Model *model) { return ((const StackModel *)model)->state == NULL; }

static size_t stack_step_weight_bytes(const CKB200Model *model)
{
    const StackModel *m = (const StackModel *)model;
    size_t s = (size_t)m->head.rows * m->head.cols;
    for (int i = 0; i < m->s.n_layers; ++i) {
        const StackLayer *l = &m->s.layers[i];
        const LinMat *list[6] = { &l->in, &l->out, &l->uq, &l->ukv, &l->a2, &l->g2 };
        for (int k = 0; k < 6; ++k) s += (size_t)list[k]->rows * list[k]->cols;
    }
    return s * 2;
}

int ckb200_model_probe_residual(CKB200Model *model, float *host_rows, int rows)
{
    if (!model || model->family != &ckb_family_stack || rows < 0) return ckb_fail(CKB_ERR_STATE, "model_probe_residual: not a layer-stack model");
    StackModel *m = (StackModel *)model;
    m->probe = rows > 0 ? host_rows : NULL;
    m->probe_rows = rows;
    m->probe_at = 0;
    return 0;
}

const CkbModelFamily ckb_family_stack = {
    .name = "layer-stack", .claims = stack_claims, .open = stack_open, .destroy = stack_destroy, .prepare = NULL, .issue_step = stack_issue_step, .extend = stack_extend,
    .clear_state = stack_clear_state, .can_set_pos = stack_can_set_pos, .step_weight_bytes = stack_step_weight_bytes,
};
