/* Weights of a layer stack: which tensors make up which stacked matrix, where the vectors lie, and filling both from a safetensors file or
 * with random numbers. */
#include <cuda_runtime_api.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#include "launch.h"
#include "mixers.h"
#include "model_stack.h"

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

static void part_name(char *dst, size_t cap, int layer, const char *prefix, const char *name)
{
    if (layer >= 0) snprintf(dst, cap, "l%d.%s%s", layer, prefix, name);
    else snprintf(dst, cap, "%s", name);
}

/* a tensor's rows appended to a stacked matrix, the first one at a multiple of `align`; returns it */
static int stack_rows_at(StackModel *m, LinMat *mat, int layer, const char *prefix, const char *name, int rows, int cols, int align)
{
    const int row0 = (mat->rows + align - 1) / align * align;
    MatPart *p = mat_part(m, mat, rows, cols, row0, 0, -1);
    if (!p) return row0;
    part_name(p->name, sizeof p->name, layer, prefix, name);
    mat->rows = row0 + pad32(rows);
    mat->cols = max2(mat->cols, pad64(cols));
    return row0;
}

static int stack_rows(StackModel *m, LinMat *mat, int layer, const char *prefix, const char *name, int rows, int cols)
{
    return stack_rows_at(m, mat, layer, prefix, name, rows, cols, 32);
}

/* a matrix beside what the stacked matrix already has, over further columns; returns the first of them */
static int stack_cols(StackModel *m, LinMat *mat, int layer, const char *prefix, const char *name, int rows, int cols)
{
    const int col0 = mat->cols;
    MatPart *p = mat_part(m, mat, rows, cols, 0, col0, -1);
    if (!p) return col0;
    part_name(p->name, sizeof p->name, layer, prefix, name);
    mat->rows = max2(mat->rows, pad32(rows));
    mat->cols += pad64(cols);
    return col0;
}

/* gate and up rows in blocks of 16 and 16; returns the first row */
static int stack_swiglu(StackModel *m, LinMat *mat, int layer, int ff, int cols)
{
    const int row0 = mat->rows;
    for (int half = 0; half < 2; ++half) {
        MatPart *p = mat_part(m, mat, ff, cols, row0, 0, half);
        if (p) part_name(p->name, sizeof p->name, layer, "mlp.", half ? "up" : "gate");
    }
    mat->rows += (ff + 15) / 16 * 32;
    mat->cols = max2(mat->cols, pad64(cols));
    return row0;
}

static VecPart *vec_part(StackModel *m, float **dst, int layer, const char *prefix, const char *name, int n, int init)
{
    VecPart *grown = (VecPart *)realloc(m->vecs, (size_t)(m->n_vecs + 1) * sizeof(VecPart));
    if (!grown) return NULL;
    m->vecs = grown;
    VecPart *p = &m->vecs[m->n_vecs++];
    memset(p, 0, sizeof *p);
    p->dst = dst;
    p->n = p->space = n;
    p->init = init;
    part_name(p->name, sizeof p->name, layer, prefix, name);
    return p;
}
/* numbers that the host has made */
static void vec_host(StackModel *m, float **dst, int layer, const char *prefix, const char *name, int n, const float *host)
{
    VecPart *p = vec_part(m, dst, layer, prefix, name, n, VEC_ONE);
    if (p) p->host = host;
}

static void plan_mixer(StackModel *m, StackLayer *l, StackMixer *x, int i)
{
    const int D = m->s.width, H = x->heads, G = x->kv_heads, ov = H * x->vdim;
    const char *px = x->prefix;
    switch (x->type) {
        case STACK_RETENTION:
            x->row_q = stack_rows(m, &l->in, i, px, "q", H * x->dim, D);
            x->row_k = stack_rows(m, &l->in, i, px, "k", H * x->dim, D);
            x->row_v = stack_rows(m, &l->in, i, px, "v", ov, D);
            x->row_g = stack_rows(m, &l->in, i, px, "g", ov, D);
            break;
        case STACK_LATENT_ATTENTION:
            x->row_dq = stack_rows(m, &l->in, i, px, "dq", x->q_rank, D);
            x->row_dkv = stack_rows(m, &l->in, i, px, "dkv", x->kv_rank + x->rot_dim, D);
            stack_rows(m, &x->uq, i, px, "uq", H * (x->dim + x->rot_dim), x->q_rank);
            stack_rows(m, &x->ukv, i, px, "uk", H * x->dim, x->kv_rank);
            x->row_uv = stack_rows(m, &x->ukv, i, px, "uv", ov, x->kv_rank);
            vec_part(m, &x->q_norm, i, px, "dq.norm", x->q_rank, VEC_ONE);
            vec_part(m, &x->kv_norm, i, px, "dkv.norm", x->kv_rank, VEC_ONE);
            break;
        case STACK_CHANNEL_DELTA:
            x->row_q = stack_rows(m, &l->in, i, px, "q", G * x->dim, D);
            x->row_k = stack_rows(m, &l->in, i, px, "k", G * x->dim, D);
            x->row_v = stack_rows(m, &l->in, i, px, "v", ov, D);
            x->row_b = stack_rows(m, &l->in, i, px, "b", H, D);
            x->row_a1 = stack_rows(m, &l->in, i, px, "a1", x->a_rank, D);
            x->row_g1 = stack_rows(m, &l->in, i, px, "g1", x->g_rank, D);
            stack_rows(m, &x->a2, i, px, "a2", H * x->dim, x->a_rank);
            stack_rows(m, &x->g2, i, px, "g2", ov, x->g_rank);
            vec_part(m, &x->a_log, i, px, "A_log", H, VEC_NOISE);
            vec_part(m, &x->dt_bias, i, px, "dt_bias", H * x->dim, VEC_NOISE);
            vec_part(m, &x->head_norm, i, px, "norm", x->vdim, VEC_ONE);
            /* the three convolutions' filters are one table over all channels: their parts follow one another */
            vec_part(m, &x->conv_w, i, px, "q.conv", G * x->dim * x->taps, VEC_NOISE);
            vec_part(m, NULL, i, px, "k.conv", G * x->dim * x->taps, VEC_NOISE);
            vec_part(m, NULL, i, px, "v.conv", ov * x->taps, VEC_NOISE);
            break;
        case STACK_WINDOW_ATTENTION:
            x->row_q = stack_rows(m, &l->in, i, px, "q", H * x->dim, D);
            x->row_k = stack_rows(m, &l->in, i, px, "k", G * x->dim, D);
            x->row_v = stack_rows(m, &l->in, i, px, "v", G * x->vdim, D);
            break;
        case STACK_LIGHTNING:
            x->row_q = stack_rows(m, &l->in, i, px, "q", H * x->dim, D);
            x->row_k = stack_rows(m, &l->in, i, px, "k", H * x->dim, D);
            x->row_v = stack_rows(m, &l->in, i, px, "v", ov, D);
            x->row_g = stack_rows(m, &l->in, i, px, "g", ov, D);
            vec_part(m, &x->head_norm, i, px, "norm", ov, VEC_ONE);
            break;
        case STACK_WKV: {
            /* every projection reads a mix of its own; the short one, whose sums take longest to store, is not the last to be computed */
            static const char *const mixes[STACK_MIXES] = { "mu.w", "mu.r", "mu.k", "mu.v", "mu.g" };
            x->row_a1 = stack_rows_at(m, &l->in, i, px, "w1", x->a_rank, D, LIN_INPUT_ROWS);
            x->row_q = stack_rows_at(m, &l->in, i, px, "r", H * x->dim, D, LIN_INPUT_ROWS);
            x->row_k = stack_rows_at(m, &l->in, i, px, "k", H * x->dim, D, LIN_INPUT_ROWS);
            x->row_v = stack_rows_at(m, &l->in, i, px, "v", ov, D, LIN_INPUT_ROWS);
            x->row_g = stack_rows_at(m, &l->in, i, px, "g", ov, D, LIN_INPUT_ROWS);
            stack_rows(m, &x->a2, i, px, "w2", H * x->dim, x->a_rank);
            for (int k = 0; k < STACK_MIXES; ++k) {
                VecPart *p = vec_part(m, k ? NULL : &x->mu, i, px, mixes[k], D, VEC_NOISE);
                if (p) p->space = pad64(D);
            }
            vec_part(m, &x->dt_bias, i, px, "w0", H * x->dim, VEC_NOISE);
            vec_part(m, &x->bonus, i, px, "u", H * x->dim, VEC_NOISE);
            vec_part(m, &x->head_norm, i, px, "norm", ov, VEC_ONE);
            break;
        }
    }
    x->col = stack_cols(m, &l->out, i, px, "o", D, ov);
}

static void plan_layer(StackModel *m, int i)
{
    StackLayer *l = &m->s.layers[i];
    const int D = m->s.width, parallel = m->s.form == STACK_PARALLEL;
    vec_part(m, &l->norm1, i, "", "norm1", D, VEC_ONE);
    for (int k = 0; k < l->arms; ++k) plan_mixer(m, l, &l->mix[k], i);
    l->z_width = l->in.rows;
    l->col_ff = l->out.cols;
    if (!l->ff) return;
    l->row_ff = stack_swiglu(m, parallel ? &l->in : &l->ff_in, i, l->ff, D);
    stack_cols(m, parallel ? &l->out : &l->ff_out, i, "mlp.", "down", D, l->ff);
    if (!parallel) vec_part(m, &l->norm2, i, "", "norm2", D, VEC_ONE);
}

#define LAYER_MATS (4 + 4 * STACK_ARMS)
/* every matrix of the model, in arena order */
static int each_mat(StackModel *m, int k, LinMat **out)
{
    if (k == 0) { *out = &m->embed; return 1; }
    if (k == 1) { *out = &m->head; return 1; }
    k -= 2;
    if (k >= LAYER_MATS * m->s.n_layers) return 0;
    StackLayer *l = &m->s.layers[k / LAYER_MATS];
    LinMat *list[LAYER_MATS] = { &l->in, &l->out, &l->ff_in, &l->ff_out };
    for (int a = 0; a < STACK_ARMS; ++a) {
        StackMixer *x = &l->mix[a];
        LinMat *of[4] = { &x->uq, &x->ukv, &x->a2, &x->g2 };
        memcpy(list + 4 + 4 * a, of, sizeof of);
    }
    *out = list[k % LAYER_MATS];
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

/* low ranks that only the tensors tell */
int ckb_stack_ranks_from_tensors(StackModel *m, const CkbSafetensors *st)
{
    for (int i = 0; i < m->s.n_layers; ++i) {
        for (int a = 0; a < m->s.layers[i].arms; ++a) {
            StackMixer *x = &m->s.layers[i].mix[a];
            const char *const names[2] = { x->type == STACK_CHANNEL_DELTA ? "a1" : (x->type == STACK_WKV ? "w1" : NULL), x->type == STACK_CHANNEL_DELTA ? "g1" : NULL };
            int *const ranks[2] = { &x->a_rank, &x->g_rank };
            for (int k = 0; k < 2; ++k) {
                if (!names[k]) continue;
                if (!st) {
                    if (*ranks[k] <= 0) *ranks[k] = k ? x->vdim : x->dim;
                    continue;
                }
                char name[64];
                CkbStTensor t;
                snprintf(name, sizeof name, "l%d.%s%s", i, x->prefix, names[k]);
                if (!ckb_st_find(st, name, &t) || t.ndim != 2 || t.shape[0] < 1 || t.shape[0] > 65536) return ckb_fail(CKB_ERR_STATE, "model: no tensor '%s'", name);
                *ranks[k] = (int)t.shape[0];
            }
        }
    }
    return 0;
}

static int fill_arena(StackModel *m, const CkbSafetensors *st, unsigned long long seed)
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
        cur += (size_t)m->vecs[i].space * sizeof(float);
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

int ckb_stack_place_weights(StackModel *m, const CkbSafetensors *st, unsigned long long seed)
{
    const StackConfig *s = &m->s;
    int rc = 0;
    float **freq = (float **)calloc((size_t)s->n_layers * STACK_ARMS, sizeof(float *));
    if (!freq) return ckb_fail(CKB_ERR_STATE, "model: out of memory");
    stack_rows(m, &m->embed, -1, "", "embed", s->vocab, s->width);
    if (!s->tied) stack_rows(m, &m->head, -1, "", "head", s->vocab, s->width);
    vec_part(m, &m->final_norm, -1, "", "final.norm", s->width, VEC_ONE);
    for (int i = 0; i < s->n_layers && !rc; ++i) {
        StackLayer *l = &s->layers[i];
        plan_layer(m, i);
        for (int a = 0; a < l->arms && !rc; ++a) {
            StackMixer *x = &l->mix[a];
            if (x->decay_host) vec_host(m, &x->decay, i, x->prefix, "decay", x->heads, x->decay_host);
            x->rot_mul = 1.0f;
            if (!x->rot_dims) continue;
            float *f = freq[i * STACK_ARMS + a] = (float *)malloc((size_t)(x->rot_dims / 2) * sizeof(float));
            if (!f) { rc = ckb_fail(CKB_ERR_STATE, "model: out of memory"); break; }
            x->rot_mul = ckb_stack_frequencies(x, f);
            vec_host(m, &x->freq, i, x->prefix, "freq", x->rot_dims / 2, f);
        }
    }
    if (!rc) rc = fill_arena(m, st, seed);
    if (!rc && s->tied) m->head = m->embed;
    for (int i = 0; i < s->n_layers * STACK_ARMS; ++i) free(freq[i]);
    free(freq);
    return rc;
}

/* what one step reads */
size_t ckb_stack_weight_elements(const StackModel *m)
{
    size_t n = (size_t)m->head.rows * m->head.cols;
    LinMat *mat;
    for (int k = 2; each_mat((StackModel *)m, k, &mat); ++k) n += (size_t)mat->rows * mat->cols;
    return n;
}
