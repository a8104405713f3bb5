// Register layout of a recurrent state: a warp holds a few columns, its lanes RPL consecutive rows of each.
#pragma once

#include <cuda_runtime.h>
#include <stdint.h>

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

// The same rows as pairs, for the packed fp32 instructions (two fused multiply-adds each); a single row gets an idle partner.
template <int RPL>
struct RecPairs {
    static constexpr int N = RPL > 1 ? RPL / 2 : 1;
    float2 v[N];
};
template <int RPL>
__device__ __forceinline__ RecPairs<RPL> rec_pairs(const RecVec<RPL> &r)
{
    RecPairs<RPL> p;
#pragma unroll
    for (int i = 0; i < RecPairs<RPL>::N; ++i) p.v[i] = make_float2(r.v[2 * i], RPL > 1 ? r.v[(2 * i + 1) % RPL] : 0.f);
    return p;
}
__device__ __forceinline__ uint64_t rec_bits(float2 v)
{
    uint64_t b;
    asm("mov.b64 %0, {%1, %2};" : "=l"(b) : "f"(v.x), "f"(v.y));
    return b;
}
__device__ __forceinline__ float2 rec_floats(uint64_t b)
{
    float2 v;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(v.x), "=f"(v.y) : "l"(b));
    return v;
}
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c)
{
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(rec_bits(a)), "l"(rec_bits(b)), "l"(rec_bits(c)));
    return rec_floats(d);
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b)
{
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(rec_bits(a)), "l"(rec_bits(b)));
    return rec_floats(d);
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
