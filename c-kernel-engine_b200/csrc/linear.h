/* Products with bfloat16 weight matrices: y[t][n] = sum_k x[t][k] W[n][k], several matrices stacked into one, with the consumer's first
 * step in the epilogue.
 *
 * A stacked matrix has its parts at rows that are multiples of 32 (zero rows between them) and its columns padded with zeros to a
 * multiple of 64.  Each 32-row block belongs to one segment, which says where its outputs go and in what form:
 *   LIN_F32     fp32 rows
 *   LIN_ACT     rows in the activation type of the pass (the input type of the next product)
 *   LIN_SWIGLU  the block holds 16 gate rows, then the 16 up rows of the same units: silu(gate) * up, activation type
 *   LIN_ADD     added to fp32 rows (the residual stream)
 *   LIN_SILU    fp32 rows, z * sigmoid(z)
 *   LIN_TANH    rows in the activation type, tanh(z)
 *   LIN_DECAY   fp32 rows, exp(-exp(z + vec[n]))
 *   LIN_CAP     fp32 rows, cap * tanh(z / cap)
 * The segments may read different inputs: x0 is the first column of a segment's input inside a row of x.  Where x0 changes, the
 * segment starts at a multiple of LIN_INPUT_ROWS.
 */
#ifndef CKB200_LINEAR_H
#define CKB200_LINEAR_H

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

enum { LIN_F32 = 0, LIN_ACT, LIN_SWIGLU, LIN_ADD, LIN_SILU, LIN_TANH, LIN_DECAY, LIN_CAP };
#define LIN_INPUT_ROWS 128

/* Type of activation rows: fp32, bfloat16, or -n (a multiple of 8): bfloat16 whose first n rows, the lead, are two pieces each that add up to
 * 16 bits and more: every eight lead rows take sixteen, first pieces before second ones, and the others follow.  The tensor-core product
 * adds the two results, so that lead rows come out as from fp32 inputs. */
enum { ACT_BF16 = 0, ACT_F32 = 1 };
#define LIN_MAX_SEGS 8
#define LIN_GEMV_MAX_TOKENS 8      /* up to here the weights are streamed past fp32 rows; above it is a matrix product */

typedef struct {
    int row0;       /* first row of the segment in the stacked matrix (a multiple of 32) */
    int count;      /* outputs per token (LIN_SWIGLU: units, twice as many rows) */
    int kind, ld;   /* ld: elements between the outputs of consecutive tokens */
    void *dst;
    int x0;
    float cap;
    const float *vec;       /* [count] */
} LinSeg;

typedef struct {
    int n;
    int act;        /* activation type */
    LinSeg s[LIN_MAX_SEGS];
} LinSegs;

typedef struct {
    const void *w;          /* bfloat16 [rows][cols] */
    int rows, cols;         /* multiples of 32 and 64 */
    uint64_t tmap[16];      /* tensor map of w (128 bytes), encoded when the matrix is placed */
} LinMat;

/* x: fp32 [tokens][ldx], at most LIN_GEMV_MAX_TOKENS rows, `cols` elements read.  norm_w (may be NULL): the input is the RMS norm of
 * the row's first norm_n elements, times norm_w (fp32), zero beyond. */
int ckb_launch_linear_gemv(const LinMat *w, const float *x, int ldx, int tokens, const float *norm_w, int norm_n, float eps, const LinSegs *segs, void *stream);

/* Input rows of the streaming product that are finished on the way in.  Rows of n elements, padded with zeros to the columns of the
 * matrix; the steps apply in this order, each only where its pointer is set. */
typedef struct {
    const float *x;
    int ldx, n;
    float eps;
    const float *y, *y_w;   /* x + RMS(y) * y_w: a sublayer's output joins the residual stream ... */
    int ldy;
    float *x_out;           /* ... and the sum is left here (rows of ldx; not x itself, which other CTAs still read) */
    const float *mu;        /* token mixing: the input of a segment is h + (before - h) * mu[x0 / columns], rows of mu as long as the matrix has columns */
    const float *before;    /* the row of the previous token, ld_before between the rows of x */
    int ld_before;
    const float *norm_w;    /* RMS norm of the row, times norm_w */
    const float *part;      /* columns from part_col on times 1 / sqrt(sum of the row's part_n partial sums / part_width + eps) */
    int part_n, part_col, part_width;
} LinInput;
int ckb_launch_linear_gemv_in(const LinMat *w, const LinInput *in, int tokens, const LinSegs *segs, void *stream);
/* any number of fp32 rows, fp32 arithmetic */
int ckb_launch_linear_f32(const LinMat *w, const float *x, int ldx, int tokens, const LinSegs *segs, void *stream);
/* any number of bfloat16 rows (16-byte aligned, ldx a multiple of 8), with a lead if segs->act says so, on the tensor cores, fp32
 * accumulation */
int ckb_launch_linear_tc(const LinMat *w, const void *x, int ldx, int tokens, const LinSegs *segs, void *stream);
int ckb_linear_encode(LinMat *w);                                   /* fills tmap; after w, rows and cols are set */
/* bfloat16 noise of standard deviation `scale` into rows x cols of a matrix with `ld` columns (synthetic models) */
int ckb_launch_fill_bf16(void *w, long long ld, int rows, int cols, int swiglu_half, float scale, unsigned long long seed, void *stream);

#ifdef __cplusplus
}
#endif
#endif
