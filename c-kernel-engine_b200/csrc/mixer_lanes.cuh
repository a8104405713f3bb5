// Register layout of a recurrent state: a warp holds four columns, its lanes RPL consecutive rows each.
#pragma once

#include <cuda_runtime.h>

namespace ckb {

template <int RPL>
struct RecVec { float v[RPL]; };
template <int RPL>
__device__ __forceinline__ RecVec<RPL> rec_read(const float *p)
{
    RecVec<RPL> r;
    if (RPL == 1) r.v[0] = p[0];
    else if (RPL == 2) { const float2 x = *reinterpret_cast<const float2 *>(p); r.v[0] = x.x; r.v[RPL - 1] = x.y; }
    else
#pragma unroll
        for (int i = 0; i < RPL / 4; ++i) {
            const float4 x = reinterpret_cast<const float4 *>(p)[i];
            r.v[(4 * i) % RPL] = x.x; r.v[(4 * i + 1) % RPL] = x.y; r.v[(4 * i + 2) % RPL] = x.z; r.v[(4 * i + 3) % RPL] = x.w;
        }
    return r;
}

// one step of a transposing butterfly: N values in, N / 2 out; lanes with bit M set keep the upper half
template <int N>
__device__ __forceinline__ void rec_fold(float *v, int lane, int m)
{
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
        const float lo = v[i], hi = v[i + N / 2];
        v[i] = ((lane & m) ? hi : lo) + __shfl_xor_sync(~0u, (lane & m) ? lo : hi, m);
    }
}

}  // namespace ckb
