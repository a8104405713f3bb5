// Output side of the bfloat16-weight products (linear.h): segment lookup and the stores of each kind.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>

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

__device__ __forceinline__ float lin_silu(float z) { return z / (1.f + expf(-z)); }

__device__ __forceinline__ void lin_store_act(void *dst, size_t i, float v, int act_f32)
{
    if (act_f32) static_cast<float *>(dst)[i] = v;
    else static_cast<__nv_bfloat16 *>(dst)[i] = __float2bfloat16_rn(v);
}

// what the segment's kind makes of a finished sum
__device__ __forceinline__ float lin_value(const LinSeg &s, int col, float v)
{
    switch (s.kind) {
        case LIN_SILU: return lin_silu(v);
        case LIN_TANH: return tanhf(v);
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
    else if (lin_is_act(s.kind)) lin_store_act(s.dst, i, lin_value(s, col, v), sg.act_f32);
    else static_cast<float *>(s.dst)[i] = lin_value(s, col, v);
}

// unit of a gate row inside a LIN_SWIGLU segment: rows come in blocks of 16 gates and their 16 ups
__device__ __forceinline__ int lin_swiglu_unit(int row_in_seg) { return (row_in_seg >> 5) * 16 + (row_in_seg & 15); }

}  // namespace ckb
