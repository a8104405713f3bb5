// Stores of activation rows: the inputs of matrix products, fp32 or bfloat16, the latter with lead rows in two pieces (linear.h, act).
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "linear.h"

namespace ckb {

// first place of activation row `row` in the buffer
__device__ __forceinline__ size_t act_row(int row, int act)
{
    if (act >= 0) return row;
    return row < -act ? (row >> 3) * 16 + (row & 7) : row - act;
}
__device__ __forceinline__ bool act_is_lead(int row, int act) { return row < -act; }
// a number less its bfloat16
__device__ __forceinline__ float act_rest(float v) { return v - __bfloat162float(__float2bfloat16_rn(v)); }

__device__ __forceinline__ void act_store(void *dst, int row, size_t ld, size_t col, float v, int act)
{
    if (act == ACT_F32) {
        static_cast<float *>(dst)[row * ld + col] = v;
        return;
    }
    __nv_bfloat16 *d = static_cast<__nv_bfloat16 *>(dst) + act_row(row, act) * ld + col;
    *d = __float2bfloat16_rn(v);
    if (act_is_lead(row, act)) d[8 * ld] = __float2bfloat16_rn(act_rest(v));
}

__device__ __forceinline__ void act_put4(__nv_bfloat16 *d, const float4 &v)
{
    __nv_bfloat162 p[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
    *reinterpret_cast<uint2 *>(d) = *reinterpret_cast<const uint2 *>(p);
}
__device__ __forceinline__ float4 act_rest4(const float4 &v) { return make_float4(act_rest(v.x), act_rest(v.y), act_rest(v.z), act_rest(v.w)); }
__device__ __forceinline__ void act_store4(void *dst, int row, size_t ld, size_t col, const float4 &v, int act)
{
    if (act == ACT_F32) {
        *reinterpret_cast<float4 *>(static_cast<float *>(dst) + row * ld + col) = v;
        return;
    }
    __nv_bfloat16 *d = static_cast<__nv_bfloat16 *>(dst) + act_row(row, act) * ld + col;
    act_put4(d, v);
    if (act_is_lead(row, act)) act_put4(d + 8 * ld, act_rest4(v));
}

}  // namespace ckb
