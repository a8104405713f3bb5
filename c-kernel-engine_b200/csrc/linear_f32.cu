// y = x W^T in fp32 arithmetic for any number of fp32 rows (weights are bfloat16 numbers, exact in fp32): 64 weight rows x 64 tokens per
// CTA, 16 columns a step, 4 x 4 outputs a thread.  The product of a model that runs in 32-bit.
#include "device_common.cuh"
#include "launch.h"
#include "linear_epilogue.cuh"
#include "runtime.h"

namespace ckb {

constexpr int LF_T = 64, LF_K = 16;

__global__ __launch_bounds__(256) void linear_f32_kernel(const __nv_bfloat16 *w, const float *x, int rows, int cols, int ldx, int tokens,
                                                         const __grid_constant__ LinSegs segs)
{
    __shared__ __align__(16) float ws[LF_K][LF_T + 4], xs[LF_K][LF_T + 4];
    __shared__ float out[LF_T][LF_T + 1];                 // [token][row]
    const int r0 = blockIdx.x * LF_T, t0 = blockIdx.y * LF_T, tr = threadIdx.x & 15, tt = threadIdx.x >> 4;
    const int in = lin_find(segs, r0);
    if (in >= 0) x += segs.s[in].x0;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < cols; k0 += LF_K) {
        for (int i = threadIdx.x; i < LF_T * LF_K; i += 256) {
            const int r = i >> 4, k = i & 15;
            ws[k][r] = r0 + r < rows ? __bfloat162float(w[(size_t)(r0 + r) * cols + k0 + k]) : 0.f;
            xs[k][r] = t0 + r < tokens ? x[(size_t)(t0 + r) * ldx + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < LF_K; ++k) {
            const float4 a = *reinterpret_cast<const float4 *>(&ws[k][tr * 4]), b = *reinterpret_cast<const float4 *>(&xs[k][tt * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) out[tt * 4 + j][tr * 4 + i] = acc[i][j];
    __syncthreads();
    for (int i = threadIdx.x; i < LF_T * LF_T; i += 256) {
        const int r = i & 63, t = i >> 6, row = r0 + r;
        if (row >= rows || t0 + t >= tokens) continue;
        const int seg = lin_find(segs, row & ~31);
        if (seg < 0) continue;
        const LinSeg &s = segs.s[seg];
        if (s.kind == LIN_SWIGLU) {
            if (row & 16) continue;
            const int unit = lin_swiglu_unit(row - s.row0);
            if (unit < s.count) act_store(s.dst, t0 + t, s.ld, unit, lin_silu(out[t][r]) * out[t][r + 16], segs.act);
        } else {
            lin_store(segs, s, t0 + t, row - s.row0, out[t][r]);
        }
    }
}

}  // namespace ckb

using namespace ckb;

extern "C" int ckb_launch_linear_f32(const LinMat *w, const float *x, int ldx, int tokens, const LinSegs *segs, void *stream)
{
    if (w->rows % 32 || w->cols % 64) return ckb_fail(CKB_ERR_SHAPE, "linear_f32: %d x %d", w->rows, w->cols);
    linear_f32_kernel<<<dim3((w->rows + LF_T - 1) / LF_T, (tokens + LF_T - 1) / LF_T), 256, 0, ckb_stream(stream)>>>(
        static_cast<const __nv_bfloat16 *>(w->w), x, w->rows, w->cols, ldx, tokens, *segs);
    return ckb_check_launch("linear_f32");
}
