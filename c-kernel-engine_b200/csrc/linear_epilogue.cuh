// Output side of the bfloat16-weight products (linear.h): segment lookup and the stores of each kind.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "act_rows.cuh"
#include "linear.h"

namespace ckb {

// segment of a row block (row0 a multiple of 32); -1 for padding rows past the last segment
__device__ __forceinline__ int lin_find(const LinSegs &sg, int row)
{
    int f = -1;
#pragma unroll
    for (int i = 0; i < LIN_MAX_SEGS; ++i)
        if (i < sg.n && row >= sg.s[i].row0) f = i;
    return f;
}

__device__ __forceinline__ float lin_silu(float z) { return __fdividef(z, 1.f + expf(-z)); }       // an infinite divisor gives 0

// 1 - 2 / (1 + exp(2 z)): an absolute error of fp32 rounding, no branches
__device__ __forceinline__ float lin_tanh(float z) { return 1.f - __fdividef(2.f, 1.f + expf(2.f * z)); }

// what the segment's kind makes of a finished sum
__device__ __forceinline__ float lin_value(const LinSeg &s, int col, float v)
{
    switch (s.kind) {
        case LIN_SILU: return lin_silu(v);
        case LIN_TANH: return lin_tanh(v);
        case LIN_DECAY: return expf(-expf(v + s.vec[col]));
        case LIN_CAP: return s.cap * tanhf(v / s.cap);
        default: return v;
    }
}
__device__ __forceinline__ bool lin_is_act(int kind) { return kind == LIN_ACT || kind == LIN_TANH; }

// one finished output of a row that is not part of a gate/up pair; col = output index inside the segment
__device__ __forceinline__ void lin_store(const LinSegs &sg, const LinSeg &s, int token, int col, float v)
{
    if (col >= s.count) return;
    const size_t i = (size_t)token * s.ld + col;
    if (s.kind == LIN_ADD) static_cast<float *>(s.dst)[i] += v;
    else if (lin_is_act(s.kind)) act_store(s.dst, token, s.ld, col, lin_value(s, col, v), sg.act);
    else static_cast<float *>(s.dst)[i] = lin_value(s, col, v);
}

// bfloat16 activation rows token, token + 1, ..: all lead rows of one block of eight, or none of them
struct LinActColumn {
    __nv_bfloat16 *d;
    size_t ld;
    bool lead;
    __device__ __forceinline__ LinActColumn(const LinSeg &s, int token, int col, int act)
        : d(static_cast<__nv_bfloat16 *>(s.dst) + act_row(token, act) * s.ld + col), ld(s.ld), lead(act_is_lead(token, act)) {}
    __device__ __forceinline__ void put(int i, float v) const
    {
        d[i * ld] = __float2bfloat16_rn(v);
        if (lead) d[(i + 8) * ld] = __float2bfloat16_rn(act_rest(v));
    }
};

// N finished sums of one output, of consecutive tokens (`tokens` of them exist), of a kind that makes something of them.  All values first:
// the functions' steps interleave.
template <int N>
__device__ __forceinline__ void lin_store_column(const LinSegs &sg, const LinSeg &s, int token, int tokens, int col, const uint32_t (&r)[N])
{
    float v[N];
    if (s.kind == LIN_SILU) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = lin_silu(__uint_as_float(r[i]));
    } else if (s.kind == LIN_DECAY) {
        const float b = s.vec[col];
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = expf(-expf(__uint_as_float(r[i]) + b));
    } else if (s.kind == LIN_TANH) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = lin_tanh(__uint_as_float(r[i]));
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = lin_value(s, col, __uint_as_float(r[i]));
    }
    if (lin_is_act(s.kind)) {
        const LinActColumn to(s, token, col, sg.act);
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (i < tokens) to.put(i, v[i]);
    } else {
        float *d = static_cast<float *>(s.dst) + (size_t)token * s.ld + col;
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (i < tokens) d[(size_t)i * s.ld] = v[i];
    }
}

// unit of a gate row inside a LIN_SWIGLU segment: rows come in blocks of 16 gates and their 16 ups
__device__ __forceinline__ int lin_swiglu_unit(int row_in_seg) { return (row_in_seg >> 5) * 16 + (row_in_seg & 15); }

}  // namespace ckb
