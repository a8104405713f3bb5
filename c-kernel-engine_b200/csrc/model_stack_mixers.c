/* The token mixers of a layer stack: their state, their projections, and their steps from the projections to the input of the output
 * projection (mixers.h has the kernels). */
#include <cuda_runtime_api.h>

#include "../../include/ckb200.h"
#include "launch.h"
#include "mixers.h"
#include "model_stack.h"
#include "runtime.h"

int ckb_stack_latent_splits(const StackModel *m, const StackMixer *x, int rows)
{
    const int groups = rows * ((x->heads + 15) / 16);
    int s = 2 * ckb_sm_count() / groups, most = (m->c.max_seq_len + 63) / 64;
    if (s > most) s = most;
    if (s > STACK_MAX_SPLITS) s = STACK_MAX_SPLITS;
    return s < 1 ? 1 : s;
}

int ckb_stack_plan_state(StackModel *m)
{
    const size_t B = (size_t)m->c.batch, eb = m->f32 ? 4 : 2;
    size_t fl = 0, cb = 0;
    m->ld_x = m->ld_h = pad64(m->s.width);
    for (int i = 0; i < m->s.n_layers; ++i) {
        StackLayer *l = &m->s.layers[i];
        m->ld_z = max2(m->ld_z, l->z_width);
        m->ld_mf = max2(m->ld_mf, max2(l->out.cols, l->ff_out.cols));
        for (int a = 0; a < l->arms; ++a) {
            StackMixer *x = &l->mix[a];
            const int H = x->heads, G = x->kv_heads, ov = pad32(H * x->vdim);
            m->ld_o = max2(m->ld_o, ov);
            if (x->type == STACK_LATENT_ATTENTION) {
                m->ld_lr = max2(m->ld_lr, x->uq.cols);
                m->ld_y = max2(m->ld_y, x->uq.rows);
                m->qa_row = max2(m->qa_row, H * (pad64(x->kv_rank) + pad32(x->rot_dim)));
                m->part_row = max2(m->part_row, H * (x->kv_rank + 2));
                x->cache_c = (void *)(uintptr_t)cb;
                cb = up256(cb + B * m->c.max_seq_len * pad64(x->kv_rank) * eb);
                x->cache_kr = (void *)(uintptr_t)cb;
                cb = up256(cb + B * m->c.max_seq_len * pad32(x->rot_dim) * eb);
                continue;
            }
            if (x->type == STACK_WINDOW_ATTENTION) {
                /* a window needs its own positions and those of the longest pass */
                const long long all = m->c.max_seq_len, ring = (long long)x->window - 1 + m->portion;
                x->cache_cap = pad64((int)(x->window && ring < all ? ring : all));
                m->q16_row = max2(m->q16_row, H * pad8(x->dim));
                x->cache_k = (void *)(uintptr_t)cb;
                cb = up256(cb + B * G * x->cache_cap * pad8(x->dim) * eb);
                x->cache_v = (void *)(uintptr_t)cb;
                cb = up256(cb + B * G * x->cache_cap * pad8(x->vdim) * eb);
                continue;
            }
            if (x->type == STACK_CHANNEL_DELTA) {
                const size_t channels = 2 * (size_t)G * x->dim + (size_t)H * x->vdim;
                m->ld_lr = max2(m->ld_lr, x->a2.cols + x->g2.cols);
                m->ld_y = max2(m->ld_y, 2 * pad32(G * x->dim) + ov);
                m->ld_g = max2(m->ld_g, x->a2.rows + x->g2.rows);
                x->conv_state = (long long)fl;
                fl += (B * x->taps * channels + 63) / 64 * 64;
            } else if (x->type == STACK_WKV) {
                m->ld_lr = max2(m->ld_lr, x->a2.cols);
                m->ld_g = max2(m->ld_g, x->a2.rows);
                m->ld_h = STACK_MIXES * m->ld_x;
                x->before = (long long)fl;
                fl += B * m->ld_x;
            } else if (x->type == STACK_LIGHTNING) {
                m->ss_row = max2(m->ss_row, H);
            }
            x->rec_state = (long long)fl;
            fl += (B * H * x->vdim * ckb_recur_dp(x->dim) + 63) / 64 * 64;
        }
    }
    m->state_floats = fl;
    m->cache_bytes = cb;
    if (fl && ckb_check_cuda((int)cudaMalloc((void **)&m->state, fl * 4), "cudaMalloc(state)")) return CKB_ERR_CUDA;
    if (fl && ckb_check_cuda((int)cudaMemset(m->state, 0, fl * 4), "zero state")) return CKB_ERR_CUDA;
    if (cb && ckb_check_cuda((int)cudaMalloc((void **)&m->cache, cb), "cudaMalloc(cache)")) return CKB_ERR_CUDA;
    if (cb && ckb_check_cuda((int)cudaMemset(m->cache, 0, cb), "zero cache")) return CKB_ERR_CUDA;
    for (int i = 0; i < m->s.n_layers; ++i)
        for (int a = 0; a < m->s.layers[i].arms; ++a) {
            StackMixer *x = &m->s.layers[i].mix[a];
            if (x->type == STACK_LATENT_ATTENTION) {
                x->cache_c = m->cache + (uintptr_t)x->cache_c;
                x->cache_kr = m->cache + (uintptr_t)x->cache_kr;
            } else if (x->type == STACK_WINDOW_ATTENTION) {
                x->cache_k = m->cache + (uintptr_t)x->cache_k;
                x->cache_v = m->cache + (uintptr_t)x->cache_v;
            }
        }
    return 0;
}

/* ------------------------------------------------------------------ projections */

/* y = W x for the rows of a pass; x in the pass's activation type */
int ckb_stack_product(const LinMat *w, const void *x, int ldx, int rows, const LinSegs *sg, void *st)
{
    if (rows <= LIN_GEMV_MAX_TOKENS) return ckb_launch_linear_gemv(w, (const float *)x, ldx, rows, NULL, 0, 0.f, sg, st);
    return sg->act == ACT_F32 ? ckb_launch_linear_f32(w, (const float *)x, ldx, rows, sg, st) : ckb_launch_linear_tc(w, x, ldx, rows, sg, st);
}

/* where the projections inside `in` go */
void ckb_stack_in_segments(const StackModel *m, const StackLayer *l, const Pass *p, LinSegs *sg)
{
    float *z = p->b->z;
    const int ld = m->ld_z, Dp = m->ld_x;
    for (int a = 0; a < l->arms; ++a) {
        const StackMixer *x = &l->mix[a];
        const int H = x->heads, G = x->kv_heads, ov = H * x->vdim;
        switch (x->type) {
            case STACK_RETENTION:
                seg_add(sg, x->row_q, H * x->dim, LIN_F32, z + x->row_q, ld);
                seg_add(sg, x->row_k, H * x->dim, LIN_F32, z + x->row_k, ld);
                seg_add(sg, x->row_v, ov, LIN_F32, z + x->row_v, ld);
                seg_add(sg, x->row_g, ov, LIN_F32, z + x->row_g, ld);
                break;
            case STACK_LATENT_ATTENTION:
                seg_add(sg, x->row_dq, x->q_rank, LIN_F32, z + x->row_dq, ld);
                seg_add(sg, x->row_dkv, x->kv_rank + x->rot_dim, LIN_F32, z + x->row_dkv, ld);
                break;
            case STACK_CHANNEL_DELTA:
                seg_add(sg, x->row_q, G * x->dim, LIN_F32, z + x->row_q, ld);
                seg_add(sg, x->row_k, G * x->dim, LIN_F32, z + x->row_k, ld);
                seg_add(sg, x->row_v, ov, LIN_F32, z + x->row_v, ld);
                seg_add(sg, x->row_b, H, LIN_F32, z + x->row_b, ld);
                seg_add(sg, x->row_a1, x->a_rank, LIN_ACT, p->b->lr, m->ld_lr);
                seg_add(sg, x->row_g1, x->g_rank, LIN_ACT, act_at(p, p->b->lr, x->a2.cols), m->ld_lr);
                break;
            case STACK_WINDOW_ATTENTION:
                seg_add(sg, x->row_q, H * x->dim, LIN_F32, z + x->row_q, ld);
                seg_add(sg, x->row_k, G * x->dim, LIN_F32, z + x->row_k, ld);
                seg_add(sg, x->row_v, G * x->vdim, LIN_F32, z + x->row_v, ld);
                break;
            case STACK_LIGHTNING:
                seg_add(sg, x->row_q, H * x->dim, LIN_SILU, z + x->row_q, ld);
                seg_add(sg, x->row_k, H * x->dim, LIN_SILU, z + x->row_k, ld);
                seg_add(sg, x->row_v, ov, LIN_SILU, z + x->row_v, ld);
                seg_add(sg, x->row_g, ov, LIN_F32, z + x->row_g, ld);
                break;
            case STACK_WKV:
                seg_from(sg, 0, x->row_a1, x->a_rank, LIN_TANH, p->b->lr, m->ld_lr);
                seg_from(sg, Dp, x->row_q, H * x->dim, LIN_F32, z + x->row_q, ld);
                seg_from(sg, 2 * Dp, x->row_k, H * x->dim, LIN_F32, z + x->row_k, ld);
                seg_from(sg, 3 * Dp, x->row_v, ov, LIN_F32, z + x->row_v, ld);
                seg_from(sg, 4 * Dp, x->row_g, ov, LIN_F32, z + x->row_g, ld);
                break;
        }
    }
}

/* ------------------------------------------------------------------ recurrent mixers */

/* one token per sequence of a mixer whose own steps are fused */
static int step_takes(const StackMixer *x, const Pass *p)
{
    if (p->T != 1 || p->act != ACT_F32 || p->R > LIN_GEMV_MAX_TOKENS || !ckb_tune_get("stack_fused_step", 1)) return 0;
    return x->type == STACK_LATENT_ATTENTION || x->type == STACK_WINDOW_ATTENTION || ckb_recur_step_takes(x->dim, x->vdim, x->a2.cols, x->g2.cols);
}

/* `ready`: the launch before this one was another mixer's step over the same projections */
static int recurrent_step(StackModel *m, const StackLayer *l, StackMixer *x, const Pass *p, int ready)
{
    const PassBuf *b = p->b;
    float *z = b->z;
    const int ld = m->ld_z;
    const RecurStep s = {
        .r = { .q = z + x->row_q, .k = z + x->row_k, .v = z + x->row_v, .ldq = ld, .ldk = ld, .ldv = ld, .decay = x->decay, .bonus = x->bonus, .G = x->kv_heads, .H = x->heads,
               .d = x->dim, .dv = x->vdim, .state = m->state + x->rec_state },
        .kind = x->type == STACK_CHANNEL_DELTA ? STEP_DELTA : (x->type == STACK_WKV ? STEP_WKV : (x->type == STACK_LIGHTNING ? STEP_LIGHTNING : STEP_RETENTION)),
        .freq = x->freq, .rot_dims = x->rot_dims, .gate = z + x->row_g, .row = p->x, .before = m->state + x->before, .row_n = m->ld_x, .ld_row = m->ld_x, .part = b->ss,
        .mul = x->out_scale, .ready = ready, .conv_w = x->conv_w, .conv_state = m->state + x->conv_state, .taps = x->taps,
        .beta = z + x->row_b, .a_low = (const float *)b->lr, .g_low = (const float *)b->lr + x->a2.cols, .a2 = x->a2.w, .g2 = x->g2.w, .ld_a2 = x->a2.cols, .ld_g2 = x->g2.cols,
        .a_log = x->a_log, .dt_bias = x->dt_bias, .head_norm = x->head_norm, .ldz = ld, .ld_low = m->ld_lr, .eps = m->s.eps, .dst = act_at(p, b->mf, x->col), .ldd = l->out.cols,
        .act_f32 = p->act == ACT_F32,
    };
    return ckb_launch_recur_step(&s, p->B, m->pos_dev, p->st);
}

static int retention_rows(StackModel *m, const StackLayer *l, StackMixer *x, const Pass *p)
{
    const PassBuf *b = p->b;
    float *z = b->z;
    const RotateRows rot[2] = {
        { .x = z + x->row_q, .ld = m->ld_z, .heads = x->heads, .head_stride = x->dim, .n = x->dim, .dims = x->rot_dims, .freq = x->freq, .mul = 1.0f },
        { .x = z + x->row_k, .ld = m->ld_z, .heads = x->heads, .head_stride = x->dim, .n = x->dim, .dims = x->rot_dims, .freq = x->freq, .mul = 1.0f / __builtin_sqrtf((float)x->dim) },
    };
    const RecurRows rec = { .q = z + x->row_q, .k = z + x->row_k, .v = z + x->row_v, .ldq = m->ld_z, .ldk = m->ld_z, .ldv = m->ld_z, .decay = x->decay, .G = x->heads,
                            .H = x->heads, .d = x->dim, .dv = x->vdim, .state = m->state + x->rec_state, .o = b->o, .ldo = m->ld_o };
    int rc = ckb_launch_rotate_rows(rot, 2, p->R, p->B, m->pos_dev, p->st);
    if (!rc) rc = ckb_launch_recur_rows(&rec, p->T, p->B, p->st);
    if (!rc) rc = ckb_launch_head_norm_gate(b->o, m->ld_o, NULL, 0, z + x->row_g, m->ld_z, GATE_SILU, m->s.eps, x->heads, x->vdim, act_at(p, b->mf, x->col), l->out.cols, p->act, p->R, p->st);
    return rc;
}

static int channel_delta_rows(StackModel *m, const StackLayer *l, StackMixer *x, const Pass *p)
{
    const PassBuf *b = p->b;
    float *z = b->z, *yq = b->y, *yk = yq + pad32(x->kv_heads * x->dim), *yv = yk + pad32(x->kv_heads * x->dim), *gate = b->g + x->a2.rows;
    LinSegs sa = { .act = p->act }, sgate = sa;
    seg_add(&sa, 0, x->heads * x->dim, LIN_F32, b->g, m->ld_g);
    seg_add(&sgate, 0, x->heads * x->vdim, LIN_F32, gate, m->ld_g);
    const ConvRows cv = { .q = z + x->row_q, .k = z + x->row_k, .v = z + x->row_v, .ld = m->ld_z, .w = x->conv_w, .state = m->state + x->conv_state, .oq = yq, .ok = yk, .ov = yv,
                          .ldo = m->ld_y, .G = x->kv_heads, .H = x->heads, .d = x->dim, .dv = x->vdim, .taps = x->taps };
    const RecurRows rec = { .q = yq, .k = yk, .v = yv, .g = b->g, .beta = z + x->row_b, .ldq = m->ld_y, .ldk = m->ld_y, .ldv = m->ld_y, .ldg = m->ld_g, .ldb = m->ld_z,
                            .G = x->kv_heads, .H = x->heads, .d = x->dim, .dv = x->vdim, .state = m->state + x->rec_state, .o = b->o, .ldo = m->ld_o };
    int rc = ckb_stack_product(&x->a2, b->lr, m->ld_lr, p->R, &sa, p->st);
    if (!rc) rc = ckb_stack_product(&x->g2, act_at(p, b->lr, x->a2.cols), m->ld_lr, p->R, &sgate, p->st);
    if (!rc) rc = ckb_launch_conv_rows(&cv, p->T, p->B, m->pos_dev, p->st);
    if (!rc) rc = ckb_launch_delta_gates(b->g, m->ld_g, x->a_log, x->dt_bias, x->heads, x->dim, z + x->row_b, m->ld_z, p->R, p->st);
    if (!rc) rc = ckb_launch_recur_rows(&rec, p->T, p->B, p->st);
    if (!rc) rc = ckb_launch_head_norm_gate(b->o, m->ld_o, x->head_norm, 0, gate, m->ld_g, GATE_SIGMOID, m->s.eps, x->heads, x->vdim, act_at(p, b->mf, x->col), l->out.cols, p->act, p->R, p->st);
    return rc;
}

static int lightning_rows(StackModel *m, const StackLayer *l, StackMixer *x, const Pass *p)
{
    const PassBuf *b = p->b;
    float *z = b->z;
    const RecurRows rec = { .q = z + x->row_q, .k = z + x->row_k, .v = z + x->row_v, .ldq = m->ld_z, .ldk = m->ld_z, .ldv = m->ld_z, .decay = x->decay, .G = x->heads,
                            .H = x->heads, .d = x->dim, .dv = x->vdim, .state = m->state + x->rec_state, .o = b->o, .ldo = m->ld_o };
    const int rc = ckb_launch_recur_rows(&rec, p->T, p->B, p->st);
    return rc ? rc : ckb_launch_row_norm_gate(b->o, m->ld_o, x->head_norm, z + x->row_g, m->ld_z, m->s.eps, x->heads * x->vdim, x->out_scale, act_at(p, b->mf, x->col), l->out.cols,
                                              p->act, p->R, p->st);
}

static int wkv_rows(StackModel *m, const StackLayer *l, StackMixer *x, const Pass *p)
{
    const PassBuf *b = p->b;
    float *z = b->z;
    LinSegs sg = { .act = p->act };
    seg_add(&sg, 0, x->heads * x->dim, LIN_DECAY, b->g, m->ld_g);
    sg.s[0].vec = x->dt_bias;
    const RecurRows rec = { .q = z + x->row_q, .k = z + x->row_k, .v = z + x->row_v, .g = b->g, .ldq = m->ld_z, .ldk = m->ld_z, .ldv = m->ld_z, .ldg = m->ld_g, .bonus = x->bonus,
                            .G = x->heads, .H = x->heads, .d = x->dim, .dv = x->vdim, .state = m->state + x->rec_state, .o = b->o, .ldo = m->ld_o };
    int rc = ckb_stack_product(&x->a2, b->lr, m->ld_lr, p->R, &sg, p->st);
    if (!rc) rc = ckb_launch_recur_rows(&rec, p->T, p->B, p->st);
    if (!rc) rc = ckb_launch_head_norm_gate(b->o, m->ld_o, x->head_norm, x->vdim, z + x->row_g, m->ld_z, GATE_SILU, m->s.eps, x->heads, x->vdim, act_at(p, b->mf, x->col), l->out.cols,
                                            p->act, p->R, p->st);
    /* the last token's input of every sequence */
    if (!rc) rc = ckb_check_cuda((int)cudaMemcpyAsync(m->state + x->before, p->x + (size_t)(p->R - p->B) * m->ld_x, (size_t)p->B * m->ld_x * 4, cudaMemcpyDeviceToDevice,
                                                      (cudaStream_t)p->st), "previous input");
    return rc;
}

/* ------------------------------------------------------------------ softmax attention over a key/value cache */

static int window_rows(StackModel *m, const StackLayer *l, StackMixer *x, const Pass *p)
{
    const PassBuf *b = p->b;
    const float *q = b->z + x->row_q, *k = b->z + x->row_k, *v = b->z + x->row_v;
    void *dst = act_at(p, b->mf, x->col);
    const KvCache c = { .H = x->heads, .G = x->kv_heads, .dim = x->dim, .vdim = x->vdim, .kd = pad8(x->dim), .vd = pad8(x->vdim), .cap = x->cache_cap, .window = x->window,
                        .cache_f32 = m->f32, .k = x->cache_k, .v = x->cache_v, .freq = x->freq, .rot_dims = x->rot_dims, .unit = 1, .rot_mul = x->rot_mul, .eps = m->s.eps,
                        .scale = x->scale, .mul = x->out_scale };
    if (p->T == 1 && ckb_tune_get("stack_fused_step", 1)) return ckb_launch_kv_attend(&c, q, k, v, m->ld_z, dst, l->out.cols, p->act == ACT_F32, p->R, p->B, m->pos_dev, p->st);
    const int portion = p->act != ACT_F32 && p->b == &m->pre && ckb_kv_prefill_takes(&c);
    const int rc = ckb_launch_kv_append(&c, q, k, v, m->ld_z, portion ? b->q16 : NULL, p->R, p->B, m->pos_dev, p->st);
    if (rc) return rc;
    if (portion) return ckb_launch_kv_prefill(&c, b->q16, dst, l->out.cols, p->act, p->T, p->B, m->pos_dev, p->st);
    return ckb_launch_kv_attend(&c, q, NULL, NULL, m->ld_z, dst, l->out.cols, p->act == ACT_F32, p->R, p->B, m->pos_dev, p->st);
}

/* ------------------------------------------------------------------ latent attention */

static LatentCache latent_cache(const StackModel *m, const StackMixer *x)
{
    LatentCache lc = { .H = x->heads, .dim = x->dim, .rot = x->rot_dim, .vdim = x->vdim, .rank = x->kv_rank, .rank_ld = pad64(x->kv_rank), .rot_ld = pad32(x->rot_dim),
                             .cap = m->c.max_seq_len, .cache_f32 = m->f32, .c = x->cache_c, .kr = x->cache_kr, .freq = x->freq, .scale = x->scale };
    lc.q_split = ckb_latent_q_split(&lc);
    return lc;
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

static int latent_expanded(StackModel *m, const StackLayer *l, StackMixer *x, const LatentCache *lc, const Pass *p)
{
    const PassBuf *b = p->b;
    const size_t keys = (size_t)m->host_pos + p->T, kw = (size_t)x->heads * x->dim, vw = (size_t)x->heads * x->vdim, qw = (size_t)x->heads * (x->dim + x->rot_dim);
    const size_t kb = up256(keys * kw * 2), vb = up256(keys * vw * 2);
    int rc = expand_alloc(m, kb + vb + up256(p->R * qw * 2));
    if (rc) return rc;
    uint8_t *k = m->expand, *v = k + kb, *q = v + vb;
    rc = ckb_launch_latent_query(lc, b->y, m->ld_y, q, p->R, p->B, m->pos_dev, p->st);
    for (int i = 0; !rc && i < p->B; ++i) {
        LinSegs sg = { .act = ACT_BF16 };
        seg_add(&sg, 0, (int)kw, LIN_ACT, k, (int)kw);
        seg_add(&sg, x->row_uv, (int)vw, LIN_ACT, v, (int)vw);
        rc = ckb_launch_linear_tc(&x->ukv, (const uint16_t *)lc->c + (size_t)i * lc->cap * lc->rank_ld, lc->rank_ld, (int)keys, &sg, p->st);
        if (!rc) rc = ckb_launch_latent_prefill(lc, q, k, v, act_at(p, b->mf, x->col), l->out.cols, p->T, p->B, i, m->pos_dev, p->st);
    }
    return rc;
}

static int latent_rows(StackModel *m, const StackLayer *l, StackMixer *x, const Pass *p)
{
    const PassBuf *b = p->b;
    const LatentCache lc = latent_cache(m, x);
    LinSegs sq = { .act = p->act };
    seg_add(&sq, 0, x->heads * (x->dim + x->rot_dim), LIN_F32, b->y, m->ld_y);
    const uint16_t *uk = (const uint16_t *)x->ukv.w, *uv = uk + (size_t)x->row_uv * x->ukv.cols;
    int rc;
    if (p->R <= LIN_GEMV_MAX_TOKENS && step_takes(x, p)) {
        const int splits = max2(1, ckb_stack_latent_splits(m, x, p->R) < b->splits ? ckb_stack_latent_splits(m, x, p->R) : b->splits);
        rc = ckb_launch_linear_gemv(&x->uq, b->z + x->row_dq, m->ld_z, p->R, x->q_norm, x->q_rank, m->s.eps, &sq, p->st);
        if (!rc) rc = ckb_launch_latent_absorb_append(&lc, b->y, m->ld_y, uk, x->ukv.cols, b->qa, b->z + x->row_dkv, m->ld_z, x->kv_norm, m->s.eps, p->R, p->B, m->pos_dev, p->st);
        if (!rc) rc = ckb_launch_latent_attend(&lc, b->qa, b->part, splits, p->R, 0, p->B, m->pos_dev, p->st);
        return rc ? rc : ckb_launch_latent_output(&lc, b->part, splits, uv, x->ukv.cols, act_at(p, b->mf, x->col), l->out.cols, p->act == ACT_F32, p->R, 0, p->B, m->pos_dev, p->st);
    }
    rc = ckb_launch_rms_rows(b->z + x->row_dq, m->ld_z, NULL, p->R, x->q_rank, x->q_norm, m->s.eps, b->lr, m->ld_lr, x->uq.cols, p->act == ACT_F32, p->st);
    if (!rc) rc = ckb_stack_product(&x->uq, b->lr, m->ld_lr, p->R, &sq, p->st);
    if (!rc) rc = ckb_launch_latent_append(&lc, b->z + x->row_dkv, m->ld_z, x->kv_norm, m->s.eps, p->R, p->B, m->pos_dev, p->st);
    if (!rc && p->act != ACT_F32 && p->b == &m->pre && ckb_latent_prefill_takes(&lc)) return latent_expanded(m, l, x, &lc, p);
    for (int r0 = 0; !rc && r0 < p->R; r0 += STACK_LATENT_ROWS) {
        const int n = p->R - r0 < STACK_LATENT_ROWS ? p->R - r0 : STACK_LATENT_ROWS;
        const int splits = max2(1, ckb_stack_latent_splits(m, x, n) < b->splits ? ckb_stack_latent_splits(m, x, n) : b->splits);
        rc = ckb_launch_latent_absorb(&lc, b->y, m->ld_y, uk, x->ukv.cols, b->qa, n, r0, p->B, m->pos_dev, p->st);
        if (!rc) rc = ckb_launch_latent_attend(&lc, b->qa, b->part, splits, n, r0, p->B, m->pos_dev, p->st);
        if (!rc) rc = ckb_launch_latent_output(&lc, b->part, splits, uv, x->ukv.cols, act_at(p, b->mf, (size_t)r0 * l->out.cols + x->col), l->out.cols, p->act == ACT_F32, n, r0, p->B, m->pos_dev, p->st);
    }
    return rc;
}

int ckb_stack_mix(StackModel *m, StackLayer *l, const Pass *p, const StackMixer **scale_rest)
{
    int rc = 0;
    *scale_rest = NULL;
    for (int a = 0; !rc && a < l->arms; ++a) {
        StackMixer *x = &l->mix[a];
        const int step = step_takes(x, p);
        switch (x->type) {
            case STACK_LATENT_ATTENTION: rc = latent_rows(m, l, x, p); break;
            case STACK_WINDOW_ATTENTION: rc = window_rows(m, l, x, p); break;
            case STACK_RETENTION: rc = step ? recurrent_step(m, l, x, p, 0) : retention_rows(m, l, x, p); break;
            case STACK_CHANNEL_DELTA: rc = step ? recurrent_step(m, l, x, p, 0) : channel_delta_rows(m, l, x, p); break;
            case STACK_WKV: rc = step ? recurrent_step(m, l, x, p, 0) : wkv_rows(m, l, x, p); break;
            case STACK_LIGHTNING:
                rc = step ? recurrent_step(m, l, x, p, a > 0 && step_takes(&l->mix[a - 1], p)) : lightning_rows(m, l, x, p);
                if (step) *scale_rest = x;
                break;
        }
    }
    return rc;
}
