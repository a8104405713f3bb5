/* Device steps of the token mixers of a layer stack (model_stack_mixers.c): rotary positions, short convolutions, linear recurrences with
 * a fixed decay, a gated delta rule or a bonus for the current token, windowed and latent attention, token mixing, gated head norms.
 * Every size and constant is a parameter.
 *
 * Rows: a pass carries T tokens of each of B sequences; row t * B + b is token t of sequence b, at position *pos + t. */
#ifndef CKB200_MIXERS_H
#define CKB200_MIXERS_H

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* x[r] = scale * table[id]; bfloat16 table with ld columns */
int ckb_launch_embed_rows(const int32_t *ids, int rows, int vocab, const void *table, int ld, int n, float scale, float *x, int ldx, void *stream);
/* dst[r] = RMS norm of src[row r, or idx[r]] * w in the activation type, zeros from n to width */
int ckb_launch_rms_rows(const float *src, int lds, const int32_t *idx, int rows, int n, const float *w, float eps, void *dst, int ldd, int width, int act_f32, void *stream);

/* Rows of the residual stream: v = x[row r, or idx[r]], plus RMS(y) * y_w where y is set, left in x_out where that is set; dst gets v, or
 * its RMS norm * norm_w, in the activation type, zeros from n to width.  With mu (no idx, no norm), dst gets n_mu mixes of v with the row
 * of the sequence's previous token instead, v + (v_before - v) * mu[i], `width` apart; the token before the pass is before[b].  x_out may
 * be x without mu only.  Every row is padded with zeros to ld, a multiple of 4. */
typedef struct {
    const float *x, *y, *y_w;
    int ldx, ldy;
    const int32_t *idx;
    float *x_out;
    const float *norm_w;
    const float *mu, *before;
    int n_mu, ld_mu, ld_before;
    void *dst;                   /* NULL: only x_out */
    int ldd, act, n, width;      /* act: activation type (linear.h) */
    float eps;
} StreamRows;
int ckb_launch_stream_rows(const StreamRows *a, int rows, int batch, void *stream);

int ckb_launch_advance_pos(int *pos, int n, void *stream);           /* *pos += n */

/* Half-split rotation of the first `dims` elements of `heads` vectors per row (head_stride apart, in place), then all n elements times mul.
 * freq: dims / 2 angular steps per position. */
typedef struct {
    float *x;
    int ld, heads, head_stride, n, dims;
    const float *freq;
    float mul;
} RotateRows;
int ckb_launch_rotate_rows(const RotateRows *a, int n_sets, int rows, int batch, const int *pos, void *stream);

/* Causal depthwise convolution over time of the channel groups q (G heads x d), k (G x d), v (H x dv), SiLU, unit length per q/k head
 * (1e-6 inside the root), q times d^-1/2.  state: ring [B][taps][channels], the input of position p in slot p % taps; the second kernel
 * stores this pass's last inputs.  Nothing before position 0 is read. */
typedef struct {
    const float *q, *k, *v;      /* projections, ld elements between rows */
    int ld;
    const float *w;              /* [channels][taps], last column on the current token */
    float *state;
    float *oq, *ok, *ov;         /* results, ldo between rows */
    int ldo, G, H, d, dv, taps;
} ConvRows;
int ckb_launch_conv_rows(const ConvRows *a, int T, int B, const int *pos, void *stream);

/* in place: decay[r][h][c] = exp(-exp(a_log[h]) * softplus(x + dt_bias[h][c])), beta = sigmoid(beta) */
int ckb_launch_delta_gates(float *decay, int ldd, const float *a_log, const float *dt_bias, int H, int d, float *beta, int ldb, int rows, void *stream);

/* Linear recurrence per head: S (d x dv) fp32, carried in `state` [B][H][dv][dp], dp = d rounded up to 32 .. 256 (ckb_recur_dp).
 *   g == NULL:      S = decay[h] S + k v^T;  o = S^T q
 *   bonus == NULL:  S = g S (per row of S); u = beta (v - S^T k); S = S + k u^T; o = S^T q
 *   else:           o = (S + diag(bonus[h]) k v^T)^T q;  S = g S + k v^T
 * q and k of head h are those of head h / (H / G). */
typedef struct {
    const float *q, *k, *v, *g, *beta;
    int ldq, ldk, ldv, ldg, ldb;
    const float *decay, *bonus;  /* [H], [H][d] */
    int G, H, d, dv;
    float *state;
    float *o;                    /* [rows][H * dv], ldo */
    int ldo;
} RecurRows;
int ckb_recur_dp(int d);         /* 0: head size not supported */
int ckb_launch_recur_rows(const RecurRows *a, int T, int B, void *stream);

/* dst[r][h * dv + i] = o / rms(o of the head) * w[h * w_stride + i] (NULL: 1) * act(gate), activation type */
enum { GATE_SILU = 0, GATE_SIGMOID = 1 };
int ckb_launch_head_norm_gate(const float *o, int ldo, const float *w, int w_stride, const float *gate, int ldg, int gate_kind, float eps, int H, int dv, void *dst, int ldd,
                              int act, int rows, void *stream);
/* dst[r][i] = o / rms(all n of the row) * w[i] * sigmoid(gate) * mul, activation type */
int ckb_launch_row_norm_gate(const float *o, int ldo, const float *w, const float *gate, int ldg, float eps, int n, float mul, void *dst, int ldd, int act, int rows, void *stream);

/* One token per sequence, everything between the two products of a recurrent mixer in one launch: rotation or convolution, gates, decay,
 * recurrence, head norm and output gate. */
enum { STEP_RETENTION = 0, STEP_DELTA, STEP_WKV, STEP_LIGHTNING };
typedef struct {
    RecurRows r;                 /* q, k, v as projected (ld* between sequences); decay of retention and lightning, bonus of wkv; the rest unused */
    int kind;
    /* all but the delta rule */
    const float *gate;           /* projected gate (SiLU; lightning: sigmoid) */
    /* retention */
    const float *freq;
    int rot_dims;
    /* wkv: low-rank input of the decay in a_low, its matrix in a2, decay = exp(-exp(a2 a_low + dt_bias)); norm weights [H * dv].  `row`
     * (row_n floats, ld_row apart) becomes `before`: the next token's previous input */
    const float *row;
    float *before;
    int row_n, ld_row;
    /* lightning: the norm spans all heads, so dst gets o * head_norm[h * dv + i] * gate * mul and part[b][h] the head's sum of squares.
     * `ready`: what the projections wrote is complete when the launch before this one lets its dependents start (that launch is then the
     * other mixer of the layer, whose results this one does not read) */
    float *part, mul;
    int ready;
    /* delta rule */
    const float *conv_w;
    float *conv_state;
    int taps;
    const float *beta, *a_low, *g_low;      /* projected beta, low-rank inputs of decay and gate (fp32) */
    const void *a2, *g2;                    /* bfloat16 [H * d][ld_a2], [H * dv][ld_g2] */
    int ld_a2, ld_g2;
    const float *a_log, *dt_bias, *head_norm;
    int ldz, ld_low;
    float eps;
    void *dst;
    int ldd, act_f32;
} RecurStep;
int ckb_recur_step_takes(int d, int dv, int ld_a2, int ld_g2);
int ckb_launch_recur_step(const RecurStep *a, int B, const int *pos, void *stream);

/* ---- softmax attention over a window, grouped queries.  A cache slab per (sequence, key head): [B][G][cap][kd] and [B][G][cap][vd], rows
 * padded with zeros to a multiple of 8; position p lives in slot p % cap, cap a multiple of 64.  A pass of T tokens overwrites no key that
 * one of its queries sees as long as T <= cap - window + 1 (window 0, all positions: as long as they fit into cap). */
typedef struct {
    int H, G, dim, vdim, kd, vd;
    int cap, window;
    int cache_f32;
    void *k, *v;
    /* query and key: the first rot_dims elements rotated (half-split) with cosines and sines times rot_mul, then `unit`: divided by the
     * root mean square over dim; scores times scale */
    const float *freq;
    int rot_dims, unit;
    float rot_mul, eps, scale;
    float mul;                   /* on the outputs */
} KvCache;
/* projected q [rows][H * dim], k [rows][G * dim], v [rows][G * vdim] (ld between rows): keys and values into the cache; q16 (may be NULL):
 * queries times scale * log2 e, bfloat16 [rows][H][kd] */
int ckb_launch_kv_append(const KvCache *c, const float *q, const float *k, const float *v, int ld, void *q16, int rows, int batch, const int *pos, void *stream);
/* Any rows over cached keys (appended before), fp32 arithmetic; k, v set: one token per sequence, appended on the way.
 * dst[r][h * vdim + i], activation type */
int ckb_launch_kv_attend(const KvCache *c, const float *q, const float *k, const float *v, int ld, void *dst, int ldd, int act_f32, int rows, int batch, const int *pos, void *stream);
/* prompt portions with a bfloat16 cache, queries from ckb_launch_kv_append, on the tensor cores */
int ckb_kv_prefill_takes(const KvCache *c);
int ckb_launch_kv_prefill(const KvCache *c, const void *q16, void *dst, int ldd, int act, int T, int batch, const int *pos, void *stream);

/* ---- latent attention: the cache holds per position the normed latent c (rank) and one rotated key part (rot) for all heads */
typedef struct {
    int H, dim, rot, vdim, rank;
    int rank_ld, rot_ld;         /* row lengths of the two caches (padded, pads zero) */
    long long cap;               /* positions per sequence */
    int cache_f32;
    int q_split;                 /* form of the absorbed queries, from ckb_latent_q_split */
    void *c, *kr;                /* [B][cap][rank_ld], [B][cap][rot_ld] */
    const float *freq;
    float scale;
} LatentCache;
/* append: kv rows [rank + rot] -> norm, rotate, store at their positions */
int ckb_launch_latent_append(const LatentCache *lc, const float *kv, int ldkv, const float *norm_w, float eps, int rows, int batch, const int *pos, void *stream);
/* Absorbed queries (scale * W_uk[h]^T q_unrotated | scale * rotated q): fp32 [r][h][rank + rot]; with q_split (a bfloat16 cache, attend on
 * the tensor cores) times log2 e as two bfloat16 pieces, [r][h][2][rank_ld + rot_ld], pads zero. */
int ckb_latent_q_split(const LatentCache *lc);
int ckb_launch_latent_absorb(const LatentCache *lc, const float *q, int ldq, const void *uk, int ld_uk, float *qa, int rows, int row0, int batch, const int *pos, void *stream);
/* absorb and append in one launch */
int ckb_launch_latent_absorb_append(const LatentCache *lc, const float *q, int ldq, const void *uk, int ld_uk, float *qa, const float *kv, int ldkv, const float *norm_w, float eps,
                                    int rows, int batch, const int *pos, void *stream);
/* softmax attention of every (row, head) over the cached latents up to the row's position, in `splits` parts:
 * part[r][h][s][rank + 2] = sum, maximum, denominator */
int ckb_launch_latent_attend(const LatentCache *lc, const float *qa, float *part, int splits, int rows, int row0, int batch, const int *pos, void *stream);
/* merge the parts and apply W_uv per head: dst[r][h * vdim + i], activation type */
int ckb_launch_latent_output(const LatentCache *lc, const float *part, int splits, const void *uv, int ld_uv, void *dst, int ldd, int act_f32, int rows, int row0, int batch,
                             const int *pos, void *stream);
/* The expanded form, for prompt portions with a bfloat16 cache and sizes that are multiples of 8: keys k [positions][H * dim] and values v
 * [positions][H * vdim] of sequence b up to the portion's end, queries from ckb_launch_latent_query ([rows][H][dim + rot], bfloat16). */
int ckb_latent_prefill_takes(const LatentCache *lc);
int ckb_launch_latent_query(const LatentCache *lc, const float *q, int ldq, void *out, int rows, int batch, const int *pos, void *stream);
int ckb_launch_latent_prefill(const LatentCache *lc, const void *q, const void *k, const void *v, void *out, int ld_out, int T, int batch, int b, const int *pos, void *stream);

#ifdef __cplusplus
}
#endif
#endif
