// Scalar functions of the mixers, fp32.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace ckb {

__device__ __forceinline__ float mix_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float mix_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float mix_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float mix_decay(float a_log, float z) { return expf(-expf(a_log) * mix_softplus(z)); }
__device__ __forceinline__ void mix_store(void *dst, size_t i, float v, int act_f32)
{
    if (act_f32) static_cast<float *>(dst)[i] = v;
    else static_cast<__nv_bfloat16 *>(dst)[i] = __float2bfloat16_rn(v);
}

}  // namespace ckb
