// y = W x for bfloat16 weights and up to eight fp32 rows: the weights are streamed once, 16 bytes a lane, past the rows in shared memory.
//
// A warp owns R weight rows at a time (for a SwiGLU segment R/2 gate rows and their up rows) and takes 256 columns a step: every lane
// eight consecutive columns of each row.  The steps of all its items form one stream that is loaded D steps ahead into registers, across
// item borders, so that loads stay in flight while an item's sums are reduced and stored.  Items are dealt to the CTAs round-robin, so
// that a matrix of few rows still occupies every SM evenly.  The rows of x sit in shared memory as two planes of 4-element groups: the two
// 16-byte reads per lane are free of bank conflicts and serve all R rows.  With a norm, the RMS factor of a row is computed while the
// row is staged, together with the norm weight, and multiplies the finished sums.  A row may also be made on the way in (LinInput): a
// sublayer's normed output added to the residual stream, mixed with the previous token's row.  Segments with inputs of their own are
// dealt to groups of CTAs in proportion to their rows, each of which stages its input only.  The first D steps of weights are fetched
// before the dependency wait of a programmatic launch.
#include "device_common.cuh"
#include "launch.h"
#include "linear_epilogue.cuh"
#include "pdl.cuh"
#include "runtime.h"

namespace ckb {


// CTAs [cta0, next cta0) take the rows [row0, row1), whose input starts at column x0
struct LinGroup { int row0, row1, cta0, x0; };
struct LinGemvParams {
    // what is read before the first weights are asked for: together, so that it takes one fetch of the parameters
    const __nv_bfloat16 *w;
    int cols, groups, rows;                // rows: end of the last group
    unsigned swiglu;                       // bit i: segment i is of that kind
    int row0[LIN_MAX_SEGS];                // first rows of the segments, past the last one beyond every row
    LinGroup g[LIN_MAX_SEGS];
    LinInput in;
    LinSegs segs;
};
__device__ __forceinline__ int lg_segment(const LinGemvParams &p, int row)      // -1: before the first
{
    int f = -1;
#pragma unroll
    for (int i = 0; i < LIN_MAX_SEGS; ++i) f += row >= p.row0[i];
    return f;
}

__device__ __forceinline__ void bf16x8_fma(const uint4 &w, const float4 &a, const float4 &b, float &acc)
{
    acc = fmaf(__uint_as_float(w.x << 16), a.x, acc);
    acc = fmaf(__uint_as_float(w.x & 0xffff0000u), a.y, acc);
    acc = fmaf(__uint_as_float(w.y << 16), a.z, acc);
    acc = fmaf(__uint_as_float(w.y & 0xffff0000u), a.w, acc);
    acc = fmaf(__uint_as_float(w.z << 16), b.x, acc);
    acc = fmaf(__uint_as_float(w.z & 0xffff0000u), b.y, acc);
    acc = fmaf(__uint_as_float(w.w << 16), b.z, acc);
    acc = fmaf(__uint_as_float(w.w & 0xffff0000u), b.w, acc);
}

// first row of a work item: R consecutive rows, or R/2 gate rows whose up rows are 16 further on
template <int R>
__device__ __forceinline__ int lg_row0(int item, bool swiglu)
{
    if (!swiglu) return item * R;
    const int per_block = 32 / R;
    return item / per_block * 32 + item % per_block * (R / 2);
}

__device__ __forceinline__ float4 lg_ld4(const float *p) { return __ldcg(reinterpret_cast<const float4 *>(p)); }

// Rows that are finished on the way in, into the two planes: x + RMS(y) y_w (JOIN), then the token mixing of the CTA's segment; with a norm
// to follow, the sums of squares go to `red` and the norm weight is multiplied in.  Elements past n are zero.  U: loads of 16 bytes per
// operand in flight.
template <int M, int WARPS, int U, bool JOIN>
__device__ __forceinline__ void lg_stream_rows(const LinGemvParams &p, int mine, float *lg_x, float (&red)[M][WARPS])
{
    constexpr int THREADS = WARPS * 32;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, groups = p.cols >> 3, n4 = p.cols >> 2;
    const LinInput &in = p.in;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float ry[M];
    if (JOIN) {
#pragma unroll
        for (int m = 0; m < M; ++m) {
            const float *yr = in.y + (size_t)m * in.ldy;
            float s = 0.f;
            for (int k0 = threadIdx.x; k0 < n4; k0 += THREADS * 4) {
                float4 y[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) y[i] = k0 + i * THREADS < n4 ? lg_ld4(yr + 4 * (k0 + i * THREADS)) : zero;
#pragma unroll
                for (int i = 0; i < 4; ++i) s = fmaf(y[i].x, y[i].x, fmaf(y[i].y, y[i].y, fmaf(y[i].z, y[i].z, fmaf(y[i].w, y[i].w, s))));
            }
            s = group_sum<32>(s);
            if (lane == 0) red[m][warp] = s;
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < M; ++m) {
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < WARPS; ++i) s += red[m][i];
            ry[m] = 1.f / sqrtf(s / (float)in.n + in.eps);
        }
        __syncthreads();                                  // `red` is written again below
    }
    const float *mu = in.mu ? in.mu + p.g[mine].x0 : nullptr;
#pragma unroll
    for (int m = 0; m < M; ++m) {
        const float *xr = in.x + (size_t)m * in.ldx, *yr = in.y + (size_t)m * in.ldy, *br = in.before + (size_t)m * in.ld_before;
        float4 *dst = reinterpret_cast<float4 *>(lg_x + (size_t)m * p.cols);
        float ss = 0.f;
        for (int k0 = threadIdx.x; k0 < n4; k0 += THREADS * U) {
            float4 v[U], y[U], w[U];
#pragma unroll
            for (int i = 0; i < U; ++i) {
                const int k = min(k0 + i * THREADS, n4 - 1) * 4;
                v[i] = lg_ld4(xr + k);
                if (JOIN) {
                    y[i] = lg_ld4(yr + k);
                    w[i] = *reinterpret_cast<const float4 *>(in.y_w + k);
                } else if (in.norm_w) {
                    w[i] = *reinterpret_cast<const float4 *>(in.norm_w + k);
                }
            }
#pragma unroll
            for (int i = 0; i < U; ++i) {
                const int k = k0 + i * THREADS;
                if (k >= n4) break;
                float4 h = v[i];
                if (4 * k + 3 >= in.n) {
                    if (4 * k >= in.n) h.x = 0.f;
                    if (4 * k + 1 >= in.n) h.y = 0.f;
                    if (4 * k + 2 >= in.n) h.z = 0.f;
                    h.w = 0.f;
                }
                if (JOIN) {
                    h.x = fmaf(y[i].x * ry[m], w[i].x, h.x); h.y = fmaf(y[i].y * ry[m], w[i].y, h.y);
                    h.z = fmaf(y[i].z * ry[m], w[i].z, h.z); h.w = fmaf(y[i].w * ry[m], w[i].w, h.w);
                    if (in.x_out && blockIdx.x == 0) reinterpret_cast<float4 *>(in.x_out + (size_t)m * in.ldx)[k] = h;
                }
                if (mu) {
                    const float4 b = lg_ld4(br + 4 * k), u = *reinterpret_cast<const float4 *>(mu + 4 * k);
                    h.x = fmaf(b.x - h.x, u.x, h.x); h.y = fmaf(b.y - h.y, u.y, h.y);
                    h.z = fmaf(b.z - h.z, u.z, h.z); h.w = fmaf(b.w - h.w, u.w, h.w);
                }
                if (in.norm_w) {
                    ss = fmaf(h.x, h.x, fmaf(h.y, h.y, fmaf(h.z, h.z, fmaf(h.w, h.w, ss))));
                    const float4 u = JOIN ? *reinterpret_cast<const float4 *>(in.norm_w + 4 * k) : w[i];
                    h.x *= u.x; h.y *= u.y; h.z *= u.z; h.w *= u.w;
                }
                dst[(k & 1) * groups + (k >> 1)] = h;
            }
        }
        if (in.norm_w) {
            ss = group_sum<32>(ss);
            if (lane == 0) red[m][warp] = ss;
        }
    }
}

// what the rows are finished with lies in memory that nothing has read since the last step: a line per thread into L2, shared out over
// the grid
__device__ __forceinline__ void lg_prefetch_vectors(const LinGemvParams &p)
{
    const int lines = p.cols / 32, line = blockIdx.x + threadIdx.x * gridDim.x;
    const LinInput &in = p.in;
    if (in.y_w && line < lines) asm volatile("prefetch.global.L2 [%0];" ::"l"(in.y_w + line * 32));
    if (in.norm_w && line < lines) asm volatile("prefetch.global.L2 [%0];" ::"l"(in.norm_w + line * 32));
    if (in.mu) {
        if (line < lines) asm volatile("prefetch.global.L2 [%0];" ::"l"(in.before + line * 32));
        if (line < p.groups * lines) asm volatile("prefetch.global.L2 [%0];" ::"l"(in.mu + line * 32));
    }
}

template <int M, int R, int D, int WARPS>
__global__ __launch_bounds__(WARPS * 32, M < 4 && WARPS == 8 ? 2 : 1) void linear_gemv_kernel(const __grid_constant__ LinGemvParams p)
{
    constexpr int LG_WARPS = WARPS, LG_THREADS = WARPS * 32;
    extern __shared__ __align__(16) float lg_x[];        // [M][2 planes][cols / 8][4]
    __shared__ float red[M][LG_WARPS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, groups = p.cols >> 3, steps = (groups + 31) >> 5;
    int mine = 0, ctas = gridDim.x, cta = blockIdx.x, items = p.rows / R, first = 0;
    if (p.groups > 1) {
#pragma unroll
        for (int i = 1; i < LIN_MAX_SEGS; ++i)
            if (i < p.groups) {
                if ((int)blockIdx.x >= p.g[i].cta0) mine = i;
                else ctas = min(ctas, p.g[i].cta0);
            }
        ctas -= p.g[mine].cta0;
        cta -= p.g[mine].cta0;
        items = p.g[mine].row1 / R;
        first = p.g[mine].row0 / R;
    }
    const int stride = ctas * LG_WARPS;
    first += warp * ctas + cta;
    // position of the next load in the warp's stream
    int l_item = first, l_g = lane;
    const __nv_bfloat16 *l_row = nullptr;
    size_t l_half = 0;                                    // from the first R/2 rows to the others
    uint4 w[D][R];
    auto enter = [&]() {
        if (l_item >= items) return;
        const int seg = lg_segment(p, l_item * R & ~31);
        const bool swiglu = seg >= 0 && (p.swiglu >> seg & 1);
        l_row = p.w + (size_t)lg_row0<R>(l_item, swiglu) * p.cols;
        l_half = (size_t)(swiglu ? 16 : R / 2) * p.cols;
    };
    auto load = [&](uint4 (&d)[R]) {
        if (l_item < items) {
            if (l_g < groups) {
#pragma unroll
                for (int i = 0; i < R; ++i) d[i] = ldg_stream_u4(l_row + (i < R / 2 ? 0 : l_half) + (size_t)(i % (R / 2)) * p.cols + l_g * 8);
            } else {
#pragma unroll
                for (int i = 0; i < R; ++i) d[i] = make_uint4(0, 0, 0, 0);
            }
            l_g += 32;
            if (l_g - lane >= groups) {
                l_g = lane;
                l_item += stride;
                enter();
            }
        }
    };
    enter();
#pragma unroll
    for (int d = 0; d < D; ++d) load(w[d]);
    lg_prefetch_vectors(p);
    pdl_wait();
    pdl_trigger();
    if (p.in.y) {
        lg_stream_rows<M, WARPS, (R * D > 12 ? 2 : 4), true>(p, mine, lg_x, red);
    } else if (p.in.mu || p.in.norm_w) {
        lg_stream_rows<M, WARPS, 4, false>(p, mine, lg_x, red);
    } else {
#pragma unroll
        for (int m = 0; m < M; ++m) {
            float scale = 1.f;                            // of the columns from part_col on
            if (p.in.part) {
                float s = 0.f;
                for (int i = lane; i < p.in.part_n; i += 32) s += __ldcg(p.in.part + (size_t)m * p.in.part_n + i);
                scale = 1.f / sqrtf(group_sum<32>(s) / (float)p.in.part_width + p.in.eps);
            }
            const float4 *xr = reinterpret_cast<const float4 *>(p.in.x + (size_t)m * p.in.ldx + p.g[mine].x0);
            float4 *dst = reinterpret_cast<float4 *>(lg_x + (size_t)m * p.cols);
            const int n = p.cols / 4;
            for (int k0 = threadIdx.x; k0 < n; k0 += LG_THREADS * 6) {
                float4 x[6];
#pragma unroll
                for (int i = 0; i < 6; ++i) x[i] = k0 + i * LG_THREADS < n ? __ldcg(xr + k0 + i * LG_THREADS) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int i = 0; i < 6; ++i) {
                    const int k = k0 + i * LG_THREADS;
                    if (p.in.part && 4 * k >= p.in.part_col) { x[i].x *= scale; x[i].y *= scale; x[i].z *= scale; x[i].w *= scale; }
                    if (k < n) dst[(k & 1) * groups + (k >> 1)] = x[i];
                }
            }
        }
    }
    __syncthreads();
    float rs[M];                                          // W (x rs) = rs (W x): the RMS factor multiplies the finished sums
#pragma unroll
    for (int m = 0; m < M; ++m) {
        rs[m] = 1.f;
        if (p.in.norm_w) {
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < LG_WARPS; ++i) ss += red[m][i];
            rs[m] = 1.f / sqrtf(ss / (float)p.in.n + p.in.eps);
        }
    }
    int item = first, step = 0;
    float acc[R][M];
#pragma unroll
    for (int i = 0; i < R; ++i)
#pragma unroll
        for (int m = 0; m < M; ++m) acc[i][m] = 0.f;
    while (item < items) {
#pragma unroll
        for (int d = 0; d < D; ++d) {
            if (item < items) {
                const int g = min(step * 32 + lane, groups - 1);
#pragma unroll
                for (int m = 0; m < M; ++m) {
                    const float4 *xs = reinterpret_cast<const float4 *>(lg_x + (size_t)m * p.cols);
                    const float4 a = xs[g], b = xs[groups + g];
#pragma unroll
                    for (int i = 0; i < R; ++i) bf16x8_fma(w[d][i], a, b, acc[i][m]);
                }
                load(w[d]);
                if (++step == steps) {
                    const int seg = lg_segment(p, item * R & ~31);
#pragma unroll
                    for (int i = 0; i < R; ++i)
#pragma unroll
                        for (int m = 0; m < M; ++m) acc[i][m] = group_sum<32>(acc[i][m]) * rs[m];
                    if (seg >= 0) {
                        // every lane holds every sum: lane (i, m) stores its own
                        const LinSeg &s = p.segs.s[seg];
                        if (s.kind == LIN_SWIGLU) {
                            const int unit0 = lin_swiglu_unit(lg_row0<R>(item, true) - s.row0);
#pragma unroll
                            for (int i = 0; i < R / 2; ++i)
#pragma unroll
                                for (int m = 0; m < M; ++m)
                                    if (lane == i * M + m && unit0 + i < s.count)
                                        act_store(s.dst, m, s.ld, unit0 + i, lin_silu(acc[i][m]) * acc[i + R / 2][m], p.segs.act);
                        } else {
#pragma unroll
                            for (int i = 0; i < R; ++i)
#pragma unroll
                                for (int m = 0; m < M; ++m)
                                    if (lane == i * M + m) lin_store(p.segs, s, m, item * R + i - s.row0, acc[i][m]);
                        }
                    }
#pragma unroll
                    for (int i = 0; i < R; ++i)
#pragma unroll
                        for (int m = 0; m < M; ++m) acc[i][m] = 0.f;
                    step = 0;
                    item += stride;
                }
            }
        }
    }
}

template <int M, int R, int D, int WARPS>
static int lg_launch(LinGemvParams p, cudaStream_t st)
{
    const size_t smem = (size_t)M * p.cols * sizeof(float);
    static size_t attr = 48 * 1024;
    if (smem > attr) {
        if (ckb_check_cuda((int)cudaFuncSetAttribute(linear_gemv_kernel<M, R, D, WARPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem), "linear_gemv smem")) return CKB_ERR_CUDA;
        attr = smem;
    }
    int per_sm = (int)((226 * 1024) / (smem + 2048));
    const int cap = M < 4 && WARPS == 8 ? 2 : 1;
    if (per_sm > cap) per_sm = cap;
    if (per_sm < 1) per_sm = 1;
    int grid = ckb_sm_count() * per_sm, rows = 0, at = 0;
    for (int i = 0; i < p.groups; ++i) rows += p.g[i].row1 - p.g[i].row0;
    if (grid > rows / R) grid = rows / R;
    // every group at least one CTA, the rest in proportion to the rows
    const int spare = grid - p.groups;
    if (spare < 0) return ckb_fail(CKB_ERR_SHAPE, "linear_gemv: %d rows for %d inputs", rows, p.groups);
    for (int i = 0, r = 0; i < p.groups; ++i) {
        p.g[i].cta0 = at + i;
        r += p.g[i].row1 - p.g[i].row0;
        at = (int)((long long)spare * r / rows);
    }
    return launch_pdl("linear_gemv", linear_gemv_kernel<M, R, D, WARPS>, dim3(grid), dim3(WARPS * 32), smem, st, p);
}

template <int M>
static int lg_pick(const LinGemvParams &p, cudaStream_t st)
{
    if constexpr (M >= 4) return lg_launch<M, 4, 2, 8>(p, st);
    // few rows: two at a time, so that every warp of the machine has work; long rows: one CTA of 16 warps per SM, x staged once for all
    else if (p.rows >= ckb_tune_get("linear_gemv_r4_rows", 16384)) return lg_launch<M, 4, 4, 8>(p, st);
    else if (p.cols >= ckb_tune_get("linear_gemv_long", 6144)) return lg_launch<M, 2, 6, 16>(p, st);
    else return lg_launch<M, 2, 6, 8>(p, st);
}

// bfloat16 noise: sum of four uniforms (variance 1/3 each after centring), scaled
__device__ __forceinline__ uint32_t lin_hash(uint64_t v)
{
    v ^= v >> 33; v *= 0xff51afd7ed558ccdull; v ^= v >> 33; v *= 0xc4ceb9fe1a85ec53ull; v ^= v >> 33;
    return (uint32_t)v;
}
__global__ void fill_bf16_kernel(__nv_bfloat16 *w, long long ld, int rows, int cols, int swiglu_half, float scale, unsigned long long seed)
{
    const long long n = (long long)rows * cols;
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const uint32_t a = lin_hash(seed * 0x9e3779b97f4a7c15ull + 2 * i), b = lin_hash(seed * 0x9e3779b97f4a7c15ull + 2 * i + 1);
        const float u = (float)(a & 0xffff) + (float)(a >> 16) + (float)(b & 0xffff) + (float)(b >> 16);
        const float v = (u * (1.f / 65536.f) - 2.f) * 1.7320508f * scale;
        long long row = i / cols;
        if (swiglu_half >= 0) row = (row >> 4) * 32 + (row & 15) + 16 * swiglu_half;
        w[row * ld + i % cols] = __float2bfloat16_rn(v);
    }
}

}  // namespace ckb

using namespace ckb;

extern "C" int ckb_launch_linear_gemv(const LinMat *w, const float *x, int ldx, int tokens, const float *norm_w, int norm_n, float eps, const LinSegs *segs, void *stream)
{
    LinInput in = {};
    in.x = x;
    in.ldx = ldx;
    in.n = norm_n;
    in.eps = eps;
    in.norm_w = norm_w;
    return ckb_launch_linear_gemv_in(w, &in, tokens, segs, stream);
}

extern "C" int ckb_launch_linear_gemv_in(const LinMat *w, const LinInput *in, int tokens, const LinSegs *segs, void *stream)
{
    if (tokens < 1 || tokens > LIN_GEMV_MAX_TOKENS || w->rows % 32 || w->cols % 64) return ckb_fail(CKB_ERR_SHAPE, "linear_gemv: %d tokens, %d x %d", tokens, w->rows, w->cols);
    if (segs->act < 0) return ckb_fail(CKB_ERR_STATE, "linear_gemv: lead rows");
    cudaStream_t st = ckb_stream(stream);
    const int fit = (int)((200 * 1024) / ((size_t)w->cols * sizeof(float)));          // rows of x that fit into shared memory
    if (fit < 1) return ckb_fail(CKB_ERR_LIMIT, "linear_gemv: rows of %d columns do not fit into shared memory", w->cols);
    for (int t = 0; t < tokens;) {
        int m = tokens - t;
        if (m > fit) m = fit;
        m = m >= 8 ? 8 : (m >= 4 ? 4 : (m >= 2 ? 2 : 1));
        LinGemvParams p = {};
        p.w = static_cast<const __nv_bfloat16 *>(w->w);
        p.cols = w->cols;
        p.in = *in;
        p.segs = *segs;
        p.in.x += (size_t)t * in->ldx;
        if (in->y) p.in.y += (size_t)t * in->ldy;
        if (in->x_out) p.in.x_out += (size_t)t * in->ldx;
        if (in->before) p.in.before += (size_t)t * in->ld_before;
        if (in->part) p.in.part += (size_t)t * in->part_n;
        p.rows = w->rows;
        for (int i = 0; i < LIN_MAX_SEGS; ++i) {
            p.row0[i] = i < segs->n ? segs->s[i].row0 : 0x7fffffff;
            if (i < segs->n && segs->s[i].kind == LIN_SWIGLU) p.swiglu |= 1u << i;
        }
        p.groups = 1;
        p.g[0].x0 = segs->s[0].x0;
        p.g[0].row1 = w->rows;
        for (int i = 1; i < segs->n; ++i) {
            if (segs->s[i].x0 == segs->s[i - 1].x0) continue;
            const LinSeg &last = segs->s[i - 1];          // a group ends with the rows that its last segment fills
            LinGroup &g = p.g[p.groups - 1], &next = p.g[p.groups++];
            g.row1 = last.row0 + (last.kind == LIN_SWIGLU ? (last.count + 15) / 16 : (last.count + 31) / 32) * 32;
            next.row0 = segs->s[i].row0;
            next.row1 = w->rows;
            next.x0 = segs->s[i].x0;
        }
        for (int i = 0; i < p.segs.n; ++i) {
            LinSeg &s = p.segs.s[i];
            const int bytes = (!(s.kind == LIN_ACT || s.kind == LIN_TANH || s.kind == LIN_SWIGLU) || segs->act == ACT_F32) ? 4 : 2;
            s.dst = static_cast<char *>(s.dst) + (size_t)t * s.ld * bytes;
        }
        const int rc = m == 8 ? lg_pick<8>(p, st) : (m == 4 ? lg_pick<4>(p, st) : (m == 2 ? lg_pick<2>(p, st) : lg_pick<1>(p, st)));
        if (rc) return rc;
        t += m;
    }
    return 0;
}

extern "C" int ckb_launch_fill_bf16(void *w, long long ld, int rows, int cols, int swiglu_half, float scale, unsigned long long seed, void *stream)
{
    fill_bf16_kernel<<<ckb_sm_count() * 8, 256, 0, ckb_stream(stream)>>>(static_cast<__nv_bfloat16 *>(w), ld, rows, cols, swiglu_half, scale, seed);
    return ckb_check_launch("fill_bf16");
}
