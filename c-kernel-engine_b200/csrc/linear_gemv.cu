// y = W x for bfloat16 weights and up to eight fp32 rows: the weights are streamed once, 16 bytes a lane, past the rows in shared memory.
//
// A warp owns R weight rows at a time (for a SwiGLU segment R/2 gate rows and their up rows) and takes 256 columns a step: every lane
// eight consecutive columns of each row.  The steps of all its items form one stream that is loaded D steps ahead into registers, across
// item borders, so that loads stay in flight while an item's sums are reduced and stored.  Items are dealt to the CTAs round-robin, so
// that a matrix of few rows still occupies every SM evenly.  The rows of x sit in shared memory as two planes of 4-element groups: the two
// 16-byte reads per lane are free of bank conflicts and serve all R rows.  With a norm, the RMS factor of a row is computed while the
// row is staged and multiplied in there, together with the norm weight.  The first D steps of weights are fetched before the dependency
// wait of a programmatic launch.
#include "device_common.cuh"
#include "launch.h"
#include "linear_epilogue.cuh"
#include "pdl.cuh"
#include "runtime.h"

namespace ckb {


struct LinGemvParams {
    const __nv_bfloat16 *w;
    const float *x, *norm_w;
    int rows, cols, ldx, norm_n;
    float eps;
    LinSegs segs;
};

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

template <int M, int R, int D, int WARPS>
__global__ __launch_bounds__(WARPS * 32, M < 4 && WARPS == 8 ? 2 : 1) void linear_gemv_kernel(const __grid_constant__ LinGemvParams p)
{
    constexpr int LG_WARPS = WARPS, LG_THREADS = WARPS * 32;
    extern __shared__ __align__(16) float lg_x[];        // [M][2 planes][cols / 8][4]
    __shared__ float red[M][LG_WARPS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, groups = p.cols >> 3, steps = (groups + 31) >> 5;
    const int items = p.rows / R, stride = gridDim.x * LG_WARPS;
    // position of the next load in the warp's stream
    int l_item = warp * gridDim.x + blockIdx.x, l_g = lane;
    const __nv_bfloat16 *l_row = nullptr;
    size_t l_half = 0;                                    // from the first R/2 rows to the others
    uint4 w[D][R];
    auto enter = [&]() {
        if (l_item >= items) return;
        const int seg = lin_find(p.segs, l_item * R & ~31);
        const bool swiglu = seg >= 0 && p.segs.s[seg].kind == LIN_SWIGLU;
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
    pdl_wait();
    pdl_trigger();
    if (p.norm_w) {
        float ss[M];
#pragma unroll
        for (int m = 0; m < M; ++m) {
            ss[m] = 0.f;
            const float *xr = p.x + (size_t)m * p.ldx;
            float *dst = lg_x + (size_t)m * p.cols;
            for (int k = threadIdx.x; k < p.cols; k += LG_THREADS) {
                const float v = k < p.norm_n ? __ldcg(xr + k) : 0.f;
                ss[m] = fmaf(v, v, ss[m]);
                dst[((k >> 2 & 1) * groups + (k >> 3)) * 4 + (k & 3)] = k < p.norm_n ? v * p.norm_w[k] : 0.f;
            }
            ss[m] = group_sum<32>(ss[m]);
            if (lane == 0) red[m][warp] = ss[m];
        }
    } else {
#pragma unroll
        for (int m = 0; m < M; ++m) {
            const float4 *xr = reinterpret_cast<const float4 *>(p.x + (size_t)m * p.ldx);
            float4 *dst = reinterpret_cast<float4 *>(lg_x + (size_t)m * p.cols);
            const int n = p.cols / 4;
            for (int k0 = threadIdx.x; k0 < n; k0 += LG_THREADS * 6) {
                float4 x[6];
#pragma unroll
                for (int i = 0; i < 6; ++i) x[i] = k0 + i * LG_THREADS < n ? __ldcg(xr + k0 + i * LG_THREADS) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int i = 0; i < 6; ++i) {
                    const int k = k0 + i * LG_THREADS;
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
        if (p.norm_w) {
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < LG_WARPS; ++i) ss += red[m][i];
            rs[m] = 1.f / sqrtf(ss / (float)p.norm_n + p.eps);
        }
    }
    int item = warp * gridDim.x + blockIdx.x, step = 0;
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
                    const int seg = lin_find(p.segs, item * R & ~31);
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
                                        lin_store_act(s.dst, (size_t)m * s.ld + unit0 + i, lin_silu(acc[i][m]) * acc[i + R / 2][m], p.segs.act_f32);
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
static int lg_launch(const LinGemvParams &p, cudaStream_t st)
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
    int grid = ckb_sm_count() * per_sm;
    if (grid > p.rows / R) grid = p.rows / R;
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
    if (tokens < 1 || tokens > LIN_GEMV_MAX_TOKENS || w->rows % 32 || w->cols % 64) return ckb_fail(CKB_ERR_SHAPE, "linear_gemv: %d tokens, %d x %d", tokens, w->rows, w->cols);
    cudaStream_t st = ckb_stream(stream);
    const int fit = (int)((200 * 1024) / ((size_t)w->cols * sizeof(float)));          // rows of x that fit into shared memory
    if (fit < 1) return ckb_fail(CKB_ERR_LIMIT, "linear_gemv: rows of %d columns do not fit into shared memory", w->cols);
    for (int t = 0; t < tokens;) {
        int m = tokens - t;
        if (m > fit) m = fit;
        m = m >= 8 ? 8 : (m >= 4 ? 4 : (m >= 2 ? 2 : 1));
        LinGemvParams p = {static_cast<const __nv_bfloat16 *>(w->w), x + (size_t)t * ldx, norm_w, w->rows, w->cols, ldx, norm_n, eps, *segs};
        for (int i = 0; i < p.segs.n; ++i) {
            LinSeg &s = p.segs.s[i];
            const int bytes = (s.kind == LIN_F32 || s.kind == LIN_ADD || segs->act_f32) ? 4 : 2;
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
