/* The family of layer-stack decoders: a folder with config.json (layer_stack_config.c) and a bfloat16 model.safetensors, or
 * "synthetic:<path of a config.json>[:seed]" with random weights of those sizes.
 *
 * Everything of a layer that reads the same input is one stacked matrix (`in`: the mixer's projections), everything that is added up is
 * another (`out`: the output projections side by side over the mixers' outputs), so a layer is products around the mixer's own steps
 * (mixers.h).  In a parallel layer, x += mixer(h) + ff(h) with h = norm(x), the feed-forward's gate and up rows belong to `in` (SwiGLU
 * in the epilogue) and its down projection to `out`, which adds to the residual in the epilogue.  In a layer with output norms,
 * x += norm1(mixer(x)), x += norm2(ff(x)), a sublayer's output waits in rows of its own until the next reader of x adds it on the way in
 * (Pass.join).  The residual, norms, angles, scores, gates and recurrent state are fp32; the inputs of the products are bfloat16 when
 * there are many rows, fp32 when there are few or the model runs in 32-bit (tune key model_f32 at open).
 *
 * State of a sequence: recurrent states, convolution tails and previous inputs (fp32), one latent and one rotated key part per position
 * (latent attention), keys and values of the last positions (windowed attention).  A pass carries T tokens of each of the `batch`
 * sequences; row t * batch + b. */
#include <cuda_runtime_api.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>
#include <sys/stat.h>

#include "../../include/ckb200.h"
#include "launch.h"
#include "mixers.h"
#include "model_stack.h"
#include "runtime.h"

/* ------------------------------------------------------------------ buffers */

static void pass_free(PassBuf *p)
{
    void *ptrs[] = { p->x, p->x2, p->d, p->ss, p->q16, p->z, p->y, p->g, p->o, p->qa, p->part, p->h, p->mf, p->lr };
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
    const size_t stream = m->s.form == STACK_OUTPUT_NORM ? R * m->ld_x * 4 : 0;
    p->splits = 1;
    for (int i = 0; i < m->s.n_layers; ++i)
        for (int a = 0; a < m->s.layers[i].arms; ++a)
            if (m->s.layers[i].mix[a].type == STACK_LATENT_ATTENTION) p->splits = max2(p->splits, ckb_stack_latent_splits(m, &m->s.layers[i].mix[a], (int)lat));
    struct { void **p; size_t bytes; } need[] = {
        { (void **)&p->x, R * m->ld_x * 4 }, { (void **)&p->h, R * m->ld_h * 4 }, { (void **)&p->z, R * m->ld_z * 4 }, { (void **)&p->mf, R * m->ld_mf * 4 },
        { (void **)&p->lr, R * m->ld_lr * 4 }, { (void **)&p->y, R * m->ld_y * 4 }, { (void **)&p->g, R * m->ld_g * 4 }, { (void **)&p->o, R * m->ld_o * 4 },
        { (void **)&p->x2, stream }, { (void **)&p->d, stream }, { (void **)&p->ss, R * m->ss_row * 4 }, { &p->q16, R * m->q16_row * 2 },
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

/* ------------------------------------------------------------------ a pass over T tokens of each sequence */

static Pass pass_begin(int T, int B, int act, const PassBuf *b, void *st)
{
    const Pass p = { .T = T, .B = B, .R = T * B, .act = act, .b = b, .st = st, .x = b->x, .other = b->x2 };
    return p;
}

/* x += mixer(h) + ff(h), h = norm1(x) */
static int parallel_layer(StackModel *m, StackLayer *l, Pass *p)
{
    const StackConfig *s = &m->s;
    const PassBuf *b = p->b;
    const StackMixer *rest;
    LinSegs in = { .act = p->act }, out = in;
    int rc;
    ckb_stack_in_segments(m, l, p, &in);
    if (l->ff) seg_add(&in, l->row_ff, l->ff, LIN_SWIGLU, act_at(p, b->mf, l->col_ff), l->out.cols);
    seg_add(&out, 0, s->width, LIN_ADD, p->x, m->ld_x);
    if (p->R <= LIN_GEMV_MAX_TOKENS) {
        rc = ckb_launch_linear_gemv(&l->in, p->x, m->ld_x, p->R, l->norm1, s->width, s->eps, &in, p->st);
    } else {
        rc = ckb_launch_rms_rows(p->x, m->ld_x, NULL, p->R, s->width, l->norm1, s->eps, b->h, m->ld_h, m->ld_h, p->act == ACT_F32, p->st);
        if (!rc) rc = ckb_stack_product(&l->in, b->h, m->ld_h, p->R, &in, p->st);
    }
    if (!rc) rc = ckb_stack_mix(m, l, p, &rest);
    return rc ? rc : ckb_stack_product(&l->out, b->mf, l->out.cols, p->R, &out, p->st);
}

/* the sum of x and what waits to join it has been left in the other buffer */
static void joined(Pass *p)
{
    if (!p->join) return;
    float *x = p->x;
    p->x = p->other;
    p->other = x;
    p->join = NULL;
}

static StreamRows stream_rows(const StackModel *m, const Pass *p)
{
    const StreamRows r = { .x = p->x, .y = p->join ? p->b->d : NULL, .y_w = p->join, .ldx = m->ld_x, .ldy = m->ld_x, .x_out = p->join ? p->other : NULL, .act = p->act,
                           .n = m->s.width, .width = m->ld_x, .eps = m->s.eps };
    return r;
}

/* W x over the residual as it stands, after what waits has joined it; mu: every segment over its own mix with the previous token's row */
static int stream_product(StackModel *m, const LinMat *w, const float *mu, const float *before, Pass *p, const LinSegs *sg)
{
    const int few = p->R <= LIN_GEMV_MAX_TOKENS;
    int rc;
    if (few && (!mu || p->T == 1)) {
        const LinInput in = { .x = p->x, .ldx = m->ld_x, .n = m->s.width, .eps = m->s.eps, .y = p->join ? p->b->d : NULL, .y_w = p->join, .ldy = m->ld_x,
                              .x_out = p->join ? p->other : NULL, .mu = mu, .before = before, .ld_before = m->ld_x };
        rc = ckb_launch_linear_gemv_in(w, &in, p->R, sg, p->st);
        joined(p);
        return rc;
    }
    StreamRows r = stream_rows(m, p);
    r.mu = mu;
    r.before = before;
    r.n_mu = STACK_MIXES;
    r.ld_mu = r.ld_before = m->ld_x;
    r.dst = p->b->h;
    r.ldd = mu ? STACK_MIXES * m->ld_x : m->ld_x;
    rc = ckb_launch_stream_rows(&r, p->R, p->B, p->st);
    joined(p);
    return rc ? rc : ckb_stack_product(w, p->b->h, r.ldd, p->R, sg, p->st);
}

/* x += norm1(mixer(x)); x += norm2(ff(x)): each sublayer leaves its output in b->d, to be joined by the next reader of x */
static int output_norm_layer(StackModel *m, StackLayer *l, Pass *p)
{
    const StackConfig *s = &m->s;
    const PassBuf *b = p->b;
    const StackMixer *rest, *wkv = l->mix[0].type == STACK_WKV ? &l->mix[0] : NULL;
    LinSegs in = { .act = p->act }, out = in, ff = in;
    ckb_stack_in_segments(m, l, p, &in);
    seg_add(&out, 0, s->width, LIN_F32, b->d, m->ld_x);
    int rc = stream_product(m, &l->in, wkv ? wkv->mu : NULL, wkv ? m->state + wkv->before : NULL, p, &in);
    if (!rc) rc = ckb_stack_mix(m, l, p, &rest);
    if (!rc && rest) {
        const LinInput last = { .x = (const float *)b->mf, .ldx = l->out.cols, .eps = s->eps, .part = b->ss, .part_n = rest->heads, .part_col = rest->col,
                                .part_width = rest->heads * rest->vdim };
        rc = ckb_launch_linear_gemv_in(&l->out, &last, p->R, &out, p->st);
    } else if (!rc) {
        rc = ckb_stack_product(&l->out, b->mf, l->out.cols, p->R, &out, p->st);
    }
    p->join = l->norm1;
    if (rc || !l->ff) return rc;
    seg_add(&ff, l->row_ff, l->ff, LIN_SWIGLU, b->mf, l->ff_out.cols);
    rc = stream_product(m, &l->ff_in, NULL, NULL, p, &ff);
    if (!rc) rc = ckb_stack_product(&l->ff_out, b->mf, l->ff_out.cols, p->R, &out, p->st);
    p->join = l->norm2;
    return rc;
}

static int issue_rows(StackModel *m, Pass *p, const int32_t *ids)
{
    const StackConfig *s = &m->s;
    const int probe = m->probe && m->probe_at + p->R <= m->probe_rows;
    int rc = ckb_launch_embed_rows(ids, p->R, s->vocab, m->embed.w, m->embed.cols, s->width, s->embed_scale, p->x, m->ld_x, p->st);
    for (int i = 0; !rc && i < s->n_layers; ++i) {
        rc = s->form == STACK_PARALLEL ? parallel_layer(m, &s->layers[i], p) : output_norm_layer(m, &s->layers[i], p);
        if (rc || !probe) continue;
        if (p->join) {
            const StreamRows r = stream_rows(m, p);
            rc = ckb_launch_stream_rows(&r, p->R, p->B, p->st);
            joined(p);
        }
        if (!rc) rc = ckb_check_cuda((int)cudaMemcpy2DAsync(m->probe + ((size_t)i * m->probe_rows + m->probe_at) * s->width, (size_t)s->width * 4, p->x, (size_t)m->ld_x * 4,
                                                            (size_t)s->width * 4, (size_t)p->R, cudaMemcpyDeviceToHost, (cudaStream_t)p->st), "residual probe");
    }
    if (probe) m->probe_at += p->R;
    return rc;
}

/* rows_dev: which rows of the pass (NULL: all n) */
static int issue_logits(StackModel *m, const Pass *p, const int32_t *rows_dev, int n, float *logits)
{
    const StackConfig *s = &m->s;
    const PassBuf *b = p->b;
    LinSegs sg = { .act = m->f32 || n <= LIN_GEMV_MAX_TOKENS ? ACT_F32 : ACT_BF16 };
    seg_add(&sg, 0, s->vocab, s->logit_cap > 0 ? LIN_CAP : LIN_F32, logits, s->vocab);
    sg.s[0].cap = s->logit_cap;
    if (!rows_dev && n <= LIN_GEMV_MAX_TOKENS) {
        const LinInput in = { .x = p->x, .ldx = m->ld_x, .n = s->width, .eps = s->eps, .y = p->join ? b->d : NULL, .y_w = p->join, .ldy = m->ld_x, .norm_w = m->final_norm };
        return ckb_launch_linear_gemv_in(&m->head, &in, n, &sg, p->st);
    }
    int rc;
    if (p->join) {
        StreamRows r = stream_rows(m, p);
        r.idx = rows_dev;
        r.x_out = NULL;
        r.norm_w = m->final_norm;
        r.dst = b->h;
        r.ldd = m->ld_x;
        r.act = sg.act;
        rc = ckb_launch_stream_rows(&r, n, 1, p->st);
    } else {
        rc = ckb_launch_rms_rows(p->x, m->ld_x, rows_dev, n, s->width, m->final_norm, s->eps, b->h, m->ld_x, m->ld_x, sg.act == ACT_F32, p->st);
    }
    return rc ? rc : ckb_stack_product(&m->head, b->h, m->ld_x, n, &sg, p->st);
}

static int stack_issue_step(CKB200Model *model, void *st)
{
    StackModel *m = (StackModel *)model;
    const int B = m->c.batch;
    Pass p = pass_begin(1, B, m->f32 || B <= LIN_GEMV_MAX_TOKENS ? ACT_F32 : ACT_BF16, &m->dec, st);
    int rc = issue_rows(m, &p, m->tokens_dev);
    if (!rc) rc = issue_logits(m, &p, NULL, B, m->logits);
    return rc ? rc : ckb_launch_advance_pos(m->pos_dev, 1, st);
}

static int stack_extend(CKB200Model *model, const int32_t *tokens, int count, const int32_t *want, int n_want, float *logits_host)
{
    StackModel *m = (StackModel *)model;
    const int B = m->c.batch, V = m->s.vocab;
    cudaStream_t st = ckb_stream(NULL);
    const int portion = m->portion < count ? m->portion : count;
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
        const int few = m->f32 || R <= LIN_GEMV_MAX_TOKENS, lead = !few && m->host_pos * B < m->lead && T > 1 ? m->lead : 0;
        Pass p = pass_begin(T, B, few ? ACT_F32 : -lead, R <= LIN_GEMV_MAX_TOKENS ? &m->few : &m->pre, st);
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

/* At the start of a sequence a recurrent head's state is the product of one key and one value: the read-out is that value times a number,
 * and the head norm divides the number out but for its sign.  Where the number is all but zero, rounded inputs turn the head's output
 * around, and the state carries that on.  So the first rows of a sequence go through the products of a prompt as two bfloat16 pieces
 * (linear.h): eight, or one of every sequence.  (The latent mixer's kernels and those beside it take no lead.) */
static void plan_lead(StackModel *m)
{
    int takes = 1;
    for (int i = 0; i < m->s.n_layers; ++i)
        for (int a = 0; a < m->s.layers[i].arms; ++a) {
            const int type = m->s.layers[i].mix[a].type;
            takes &= type == STACK_WKV || type == STACK_LIGHTNING || type == STACK_WINDOW_ATTENTION;
        }
    m->lead = takes && !m->f32 && ckb_tune_get("stack_lead", 1) ? pad8(m->c.batch) : 0;
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
    m->c.num_heads = m->c.num_kv_heads = sc.layers[0].mix[0].heads;
    m->c.head_dim = sc.layers[0].mix[0].dim;
    m->c.intermediate_size = sc.layers[0].ff;
    m->c.rms_eps = sc.eps;
    m->c.batch = batch > 0 ? batch : 1;
    m->c.tp_size = 1;
    m->c.max_seq_len = ckb_tune_get("model_max_seq", 4096);
    m->portion = max2(1, ckb_tune_get("stack_portion", 2048) / m->c.batch);
    int rc = m->c.max_seq_len < 1 ? ckb_fail(CKB_ERR_SHAPE, "model_max_seq: %d", m->c.max_seq_len) : 0;
    if (!rc && !synth && !(st = ckb_st_open(weights))) rc = CKB_ERR_STATE;
    if (!rc) rc = ckb_stack_ranks_from_tensors(m, st);
    if (!rc && ckb_ensure_init()) rc = CKB_ERR_NO_DEVICE;
    if (!rc) rc = ckb_stack_place_weights(m, st, seed);
    if (!rc) rc = ckb_model_init_shared((CKB200Model *)m);
    if (!rc) rc = ckb_stack_plan_state(m);
    if (!rc) plan_lead(m);
    if (!rc) rc = pass_alloc(m, &m->dec, m->c.batch);
    if (!rc) rc = ckb_check_cuda((int)cudaStreamSynchronize(ckb_stream(NULL)), "model init");
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

/* neither a recurrent state nor a window's slots can go back */
static int stack_can_set_pos(const CKB200Model *model)
{
    const StackModel *m = (const StackModel *)model;
    for (int i = 0; i < m->s.n_layers; ++i)
        for (int a = 0; a < m->s.layers[i].arms; ++a)
            if (m->s.layers[i].mix[a].type == STACK_WINDOW_ATTENTION) return 0;
    return m->state == NULL;
}

static size_t stack_step_weight_bytes(const CKB200Model *model) { return 2 * ckb_stack_weight_elements((const StackModel *)model); }

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
