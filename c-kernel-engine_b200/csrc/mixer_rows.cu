// Row-wise steps around the mixers of a layer stack: embedding, RMS norm, rotary positions, short convolutions, delta-rule gates, gated
// head norm.  One warp or CTA per row or head; everything in fp32, the activation type only where a result feeds a matrix product.
#include <cuda_bf16.h>

#include "act_rows.cuh"
#include "device_common.cuh"
#include "launch.h"
#include "mixer_math.cuh"
#include "mixers.h"
#include "pdl.cuh"
#include "runtime.h"

namespace ckb {

__global__ void embed_rows_kernel(const int32_t *ids, int vocab, const __nv_bfloat16 *table, int ld, int n, float scale, float *x, int ldx)
{
    pdl_wait();
    pdl_trigger();
    const int id = __ldcg(ids + blockIdx.x);
    for (int i = threadIdx.x; i < n; i += blockDim.x)
        x[(size_t)blockIdx.x * ldx + i] = (unsigned)id < (unsigned)vocab ? __bfloat162float(table[(size_t)id * ld + i]) * scale : 0.f;
}

__global__ __launch_bounds__(256) void rms_rows_kernel(const float *src, int lds, const int32_t *idx, int n, const float *w, float eps, void *dst, int ldd, int width, int act_f32)
{
    __shared__ float red[8];
    pdl_wait();
    pdl_trigger();
    const float *s = src + (size_t)(idx ? idx[blockIdx.x] : blockIdx.x) * lds;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += 256) { const float v = __ldcg(s + i); ss = fmaf(v, v, ss); }
    ss = group_sum<32>(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += red[i];
    const float rs = 1.f / sqrtf(ss / (float)n + eps);
    for (int i = threadIdx.x; i < width; i += 256) mix_store(dst, (size_t)blockIdx.x * ldd + i, i < n ? __ldcg(s + i) * rs * w[i] : 0.f, act_f32);
}

__device__ __forceinline__ float4 sr_ld4(const float *p) { return __ldcg(reinterpret_cast<const float4 *>(p)); }
__device__ __forceinline__ float sr_dot4(const float4 &a, float s) { return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, fmaf(a.w, a.w, s)))); }
// sum over the block's 256 threads, in every thread; `red` is free again after the next barrier
__device__ __forceinline__ float sr_block_sum(float s, float *red)
{
    s = group_sum<32>(s);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = s;
    __syncthreads();
    s = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s += red[i];
    return s;
}

// U groups of four elements per thread, in registers (width <= 1024 U)
template <int U>
__global__ __launch_bounds__(256) void stream_rows_kernel(const __grid_constant__ StreamRows a)
{
    __shared__ float red[2][8];
    pdl_wait();
    pdl_trigger();
    const int r = a.idx ? a.idx[blockIdx.x] : blockIdx.x, n4 = a.width >> 2;
    const float *xr = a.x + (size_t)r * a.ldx, *yr = a.y + (size_t)r * a.ldy;
    float4 v[U], y[U];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < U; ++i) {
        const int k = threadIdx.x + i * 256;
        v[i] = y[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (k < n4) {
            v[i] = sr_ld4(xr + 4 * k);
            if (a.y) y[i] = sr_ld4(yr + 4 * k);
        }
        s = sr_dot4(y[i], s);
    }
    if (a.y) {
        const float rs = 1.f / sqrtf(sr_block_sum(s, red[0]) / (float)a.n + a.eps);
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const int k = threadIdx.x + i * 256;
            if (k >= n4) break;
            const float4 w = *reinterpret_cast<const float4 *>(a.y_w + 4 * k);
            v[i].x = fmaf(y[i].x * rs, w.x, v[i].x); v[i].y = fmaf(y[i].y * rs, w.y, v[i].y);
            v[i].z = fmaf(y[i].z * rs, w.z, v[i].z); v[i].w = fmaf(y[i].w * rs, w.w, v[i].w);
            if (a.x_out) reinterpret_cast<float4 *>(a.x_out + (size_t)r * a.ldx)[k] = v[i];
        }
    }
    if (!a.dst) return;
    if (a.norm_w) {
        s = 0.f;
#pragma unroll
        for (int i = 0; i < U; ++i) s = sr_dot4(v[i], s);
        s = 1.f / sqrtf(sr_block_sum(s, red[1]) / (float)a.n + a.eps);
    }
#pragma unroll
    for (int i = 0; i < U; ++i) {
        const int k = threadIdx.x + i * 256;
        if (k >= n4) break;
        if (a.norm_w) {
            const float4 w = *reinterpret_cast<const float4 *>(a.norm_w + 4 * k);
            v[i].x *= s * w.x; v[i].y *= s * w.y; v[i].z *= s * w.z; v[i].w *= s * w.w;
        }
        act_store4(a.dst, blockIdx.x, a.ldd, 4 * k, v[i], a.act);
    }
}

// the same with token mixing: a CTA walks `run` tokens of one sequence, after the one before them
template <int U>
__global__ __launch_bounds__(256) void stream_mix_kernel(const __grid_constant__ StreamRows a, int T, int B, int run)
{
    __shared__ float red[2][8];
    pdl_wait();
    pdl_trigger();
    const int b = blockIdx.x % B, t0 = blockIdx.x / B * run, n4 = a.width >> 2;
    float4 last[U];
#pragma unroll
    for (int i = 0; i < U; ++i) last[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int t = t0 - 1; t < min(t0 + run, T); ++t) {
        float4 v[U];
        if (t < 0) {
#pragma unroll
            for (int i = 0; i < U; ++i)
                if (threadIdx.x + i * 256 < n4) last[i] = sr_ld4(a.before + (size_t)b * a.ld_before + 4 * (threadIdx.x + i * 256));
            continue;
        }
        const size_t r = (size_t)t * B + b;
        float4 y[U];
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const int k = threadIdx.x + i * 256;
            v[i] = y[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (k < n4) {
                v[i] = sr_ld4(a.x + r * a.ldx + 4 * k);
                if (a.y) y[i] = sr_ld4(a.y + r * a.ldy + 4 * k);
            }
            s = sr_dot4(y[i], s);
        }
        if (a.y) {
            const float rs = 1.f / sqrtf(sr_block_sum(s, red[t & 1]) / (float)a.n + a.eps);
#pragma unroll
            for (int i = 0; i < U; ++i) {
                const int k = threadIdx.x + i * 256;
                if (k >= n4) break;
                const float4 w = *reinterpret_cast<const float4 *>(a.y_w + 4 * k);
                v[i].x = fmaf(y[i].x * rs, w.x, v[i].x); v[i].y = fmaf(y[i].y * rs, w.y, v[i].y);
                v[i].z = fmaf(y[i].z * rs, w.z, v[i].z); v[i].w = fmaf(y[i].w * rs, w.w, v[i].w);
                if (a.x_out && t >= t0) reinterpret_cast<float4 *>(a.x_out + r * a.ldx)[k] = v[i];
            }
        }
        if (t >= t0) {
            const size_t at = act_row((int)r, a.act) * a.ldd;
            const bool lead = act_is_lead((int)r, a.act), f32 = a.act == ACT_F32;
#pragma unroll
            for (int i = 0; i < U; ++i) {
                const int k = threadIdx.x + i * 256;
                if (k >= n4) break;
                for (int j = 0; j < a.n_mu; ++j) {
                    const float4 w = *reinterpret_cast<const float4 *>(a.mu + (size_t)j * a.ld_mu + 4 * k);
                    const float4 x = make_float4(fmaf(last[i].x - v[i].x, w.x, v[i].x), fmaf(last[i].y - v[i].y, w.y, v[i].y), fmaf(last[i].z - v[i].z, w.z, v[i].z),
                                                 fmaf(last[i].w - v[i].w, w.w, v[i].w));
                    const size_t to = at + (size_t)j * a.width + 4 * k;
                    if (f32) {
                        *reinterpret_cast<float4 *>(static_cast<float *>(a.dst) + to) = x;
                    } else {
                        __nv_bfloat16 *d = static_cast<__nv_bfloat16 *>(a.dst) + to;
                        act_put4(d, x);
                        if (lead) act_put4(d + 8 * (size_t)a.ldd, act_rest4(x));
                    }
                }
            }
        }
#pragma unroll
        for (int i = 0; i < U; ++i) last[i] = v[i];
    }
}

__global__ void advance_pos_kernel(int *pos, int n)
{
    pdl_wait();
    pdl_trigger();
    *pos += n;
}

struct RotateSets { RotateRows s[2]; };
__global__ __launch_bounds__(256) void rotate_rows_kernel(const __grid_constant__ RotateSets sets, int batch, const int *pos)
{
    extern __shared__ float rot_cs[];                        // cosines, then sines, of this row's position
    pdl_wait();
    pdl_trigger();
    const RotateRows &a = sets.s[blockIdx.y];
    const float p = (float)(__ldcg(pos) + (int)blockIdx.x / batch);
    const int half = a.dims / 2;
    for (int i = threadIdx.x; i < half; i += 256) sincosf(p * a.freq[i], &rot_cs[half + i], &rot_cs[i]);
    __syncthreads();
    const int per = a.n - half, warp = threadIdx.x >> 5;      // per head: half pairs, then the elements that pass
    for (int h = warp; h < a.heads; h += 8) {
        float *x = a.x + (size_t)blockIdx.x * a.ld + h * a.head_stride;
        for (int j = threadIdx.x & 31; j < per; j += 32) {
            if (j < half) {
                const float c = rot_cs[j], s = rot_cs[half + j], u = x[j], v = x[j + half];
                x[j] = (u * c - v * s) * a.mul;
                x[j + half] = (v * c + u * s) * a.mul;
            } else {
                x[j + half] *= a.mul;
            }
        }
    }
}

// one warp per (head vector, CONV_TOKENS tokens of a sequence): G q heads, G k heads, H v heads; NC channels per lane
constexpr int CONV_TOKENS = 8;
template <int NC>
__global__ __launch_bounds__(128) void conv_rows_kernel(const __grid_constant__ ConvRows a, int T, int B, const int *pos)
{
    pdl_wait();
    pdl_trigger();
    const int b = blockIdx.x % B, t0 = blockIdx.x / B * CONV_TOKENS, lane = threadIdx.x & 31, nt = min(CONV_TOKENS, T - t0);
    const int vec = blockIdx.y * 4 + (threadIdx.x >> 5);
    if (vec >= 2 * a.G + a.H) return;
    const int kind = vec < a.G ? 0 : (vec < 2 * a.G ? 1 : 2);
    const int head = kind == 0 ? vec : (kind == 1 ? vec - a.G : vec - 2 * a.G), n = kind == 2 ? a.dv : a.d;
    const float *src = (kind == 0 ? a.q : (kind == 1 ? a.k : a.v)) + (size_t)b * a.ld + head * n;
    float *dst = (kind == 0 ? a.oq : (kind == 1 ? a.ok : a.ov)) + (size_t)b * a.ldo + head * n;
    const int channels = 2 * a.G * a.d + a.H * a.dv, ch0 = (kind == 0 ? 0 : (kind == 1 ? a.G * a.d : 2 * a.G * a.d)) + head * n;
    const int back = a.taps - 1, p0 = __ldcg(pos);
    const float *old = a.state + (size_t)b * a.taps * channels + ch0;
    float acc[CONV_TOKENS][NC];
#pragma unroll
    for (int t = 0; t < CONV_TOKENS; ++t)
#pragma unroll
        for (int c = 0; c < NC; ++c) acc[t][c] = 0.f;
#pragma unroll 1
    for (int j = 0; j < a.taps; ++j) {
        float w[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) w[c] = lane + 32 * c < n ? a.w[(size_t)(ch0 + lane + 32 * c) * a.taps + j] : 0.f;
#pragma unroll
        for (int t = 0; t < CONV_TOKENS; ++t) {
            const int at = t0 + t - back + j;                // time of this tap relative to the pass
            if (t >= nt || p0 + at < 0) continue;
            const float *x = at >= 0 ? src + (size_t)at * B * a.ld : old + (size_t)((p0 + at) % a.taps) * channels;
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (lane + 32 * c < n) acc[t][c] = fmaf(w[c], x[lane + 32 * c], acc[t][c]);
        }
    }
#pragma unroll
    for (int t = 0; t < CONV_TOKENS; ++t) {
        if (t >= nt) break;
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            acc[t][c] = mix_silu(acc[t][c]);                 // channels past n: silu(0) = 0
            ss = fmaf(acc[t][c], acc[t][c], ss);
        }
        const float mul = kind == 2 ? 1.f : 1.f / sqrtf(group_sum<32>(ss) + 1e-6f) * (kind == 0 ? 1.f / sqrtf((float)a.d) : 1.f);
#pragma unroll
        for (int c = 0; c < NC; ++c)
            if (lane + 32 * c < n) dst[(size_t)(t0 + t) * B * a.ldo + lane + 32 * c] = acc[t][c] * mul;
    }
}

// the inputs of the last taps - 1 tokens go into the ring
__global__ void conv_state_kernel(const __grid_constant__ ConvRows a, int T, int B, const int *pos)
{
    pdl_wait();
    pdl_trigger();
    const int channels = 2 * a.G * a.d + a.H * a.dv, c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y, p0 = __ldcg(pos);
    if (c >= channels) return;
    const float *src = c < a.G * a.d ? a.q + c : (c < 2 * a.G * a.d ? a.k + (c - a.G * a.d) : a.v + (c - 2 * a.G * a.d));
    float *s = a.state + (size_t)b * a.taps * channels + c;
    for (int t = max(0, T - (a.taps - 1)); t < T; ++t) s[(size_t)((p0 + t) % a.taps) * channels] = src[(size_t)(t * B + b) * a.ld];
}

__global__ void delta_gates_kernel(float *decay, int ldd, const float *a_log, const float *dt_bias, int H, int d, float *beta, int ldb)
{
    pdl_wait();
    pdl_trigger();
    for (int i = threadIdx.x; i < H * d; i += blockDim.x) {
        float *g = decay + (size_t)blockIdx.x * ldd + i;
        *g = mix_decay(a_log[i / d], *g + dt_bias[i]);
    }
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float *x = beta + (size_t)blockIdx.x * ldb + i;
        *x = mix_sigmoid(*x);
    }
}

__global__ __launch_bounds__(128) void head_norm_gate_kernel(const float *o, int ldo, const float *w, int w_stride, const float *gate, int ldg, int gate_kind, float eps, int H, int dv,
                                                             void *dst, int ldd, int act)
{
    pdl_wait();
    pdl_trigger();
    const int row = blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (h >= H) return;
    const float *s = o + (size_t)row * ldo + h * dv, *g = gate + (size_t)row * ldg + h * dv;
    float ss = 0.f;
    for (int i = lane; i < dv; i += 32) ss = fmaf(s[i], s[i], ss);
    const float rs = 1.f / sqrtf(group_sum<32>(ss) / (float)dv + eps);
    for (int i = lane; i < dv; i += 32)
        act_store(dst, row, ldd, h * dv + i, s[i] * rs * (w ? w[h * w_stride + i] : 1.f) * (gate_kind == GATE_SILU ? mix_silu(g[i]) : mix_sigmoid(g[i])), act);
}

// the same for heads of a multiple of four elements, at most 4 * L: L lanes per head, four heads of a lane at a time
template <int L>
__global__ __launch_bounds__(256) void head_norm_gate4_kernel(const float *o, int ldo, const float *w, int w_stride, const float *gate, int ldg, int gate_kind, float eps, int H, int dv,
                                                              void *dst, int ldd, int act)
{
    constexpr int HEADS = 256 / L, U = 4;
    pdl_wait();
    pdl_trigger();
    const int row = blockIdx.x, sub = threadIdx.x % L;
    for (int h0 = blockIdx.y * HEADS * U + threadIdx.x / L; h0 - threadIdx.x / L < H; h0 += gridDim.y * HEADS * U) {      // whole warps stay together
        float4 v[U], z[U], g[U];
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const int h = h0 + i * HEADS;
            v[i] = z[i] = g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (h < H && 4 * sub < dv) {
                v[i] = sr_ld4(o + (size_t)row * ldo + h * dv + 4 * sub);
                z[i] = sr_ld4(gate + (size_t)row * ldg + h * dv + 4 * sub);
                g[i] = w ? *reinterpret_cast<const float4 *>(w + h * w_stride + 4 * sub) : make_float4(1.f, 1.f, 1.f, 1.f);
            }
        }
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const int h = h0 + i * HEADS;
            const float rs = 1.f / sqrtf(group_sum<L>(sr_dot4(v[i], 0.f)) / (float)dv + eps);
            auto gated = [&](float x) { return gate_kind == GATE_SILU ? mix_silu(x) : mix_sigmoid(x); };
            if (h < H && 4 * sub < dv)
                act_store4(dst, row, ldd, h * dv + 4 * sub,
                          make_float4(v[i].x * rs * g[i].x * gated(z[i].x), v[i].y * rs * g[i].y * gated(z[i].y), v[i].z * rs * g[i].z * gated(z[i].z), v[i].w * rs * g[i].w * gated(z[i].w)), act);
        }
    }
}

__global__ __launch_bounds__(256) void row_norm_gate_kernel(const float *o, int ldo, const float *w, const float *gate, int ldg, float eps, int n, float mul, void *dst, int ldd, int act)
{
    __shared__ float red[8];
    pdl_wait();
    pdl_trigger();
    const float *s = o + (size_t)blockIdx.x * ldo, *g = gate + (size_t)blockIdx.x * ldg;
    float ss = 0.f;
#pragma unroll 4
    for (int i = threadIdx.x; i < n; i += 256) { const float v = __ldcg(s + i); ss = fmaf(v, v, ss); }
    const float rs = mul / sqrtf(sr_block_sum(ss, red) / (float)n + eps);
#pragma unroll 4
    for (int i = threadIdx.x; i < n; i += 256) act_store(dst, blockIdx.x, ldd, i, __ldcg(s + i) * rs * w[i] * mix_sigmoid(__ldcg(g + i)), act);
}

}  // namespace ckb

using namespace ckb;

extern "C" int ckb_launch_stream_rows(const StreamRows *a, int rows, int batch, void *stream)
{
    cudaStream_t st = ckb_stream(stream);
    const int u = (a->width + 1023) / 1024;
    if (a->width % 4 || u > 16) return ckb_fail(CKB_ERR_LIMIT, "stream_rows: width %d", a->width);
    if (a->mu) {
        const int T = rows / batch, even = (rows + 2 * ckb_sm_count() - 1) / (2 * ckb_sm_count()), run = even < 8 ? even : 8;
        const dim3 grid((T + run - 1) / run * batch);
        if (u <= 1) return launch_pdl("stream_mix", stream_mix_kernel<1>, grid, dim3(256), 0, st, *a, T, batch, run);
        if (u <= 2) return launch_pdl("stream_mix", stream_mix_kernel<2>, grid, dim3(256), 0, st, *a, T, batch, run);
        if (u <= 4) return launch_pdl("stream_mix", stream_mix_kernel<4>, grid, dim3(256), 0, st, *a, T, batch, run);
        if (u <= 8) return launch_pdl("stream_mix", stream_mix_kernel<8>, grid, dim3(256), 0, st, *a, T, batch, run);
        return launch_pdl("stream_mix", stream_mix_kernel<16>, grid, dim3(256), 0, st, *a, T, batch, run);
    }
    if (u <= 1) return launch_pdl("stream_rows", stream_rows_kernel<1>, dim3(rows), dim3(256), 0, st, *a);
    if (u <= 2) return launch_pdl("stream_rows", stream_rows_kernel<2>, dim3(rows), dim3(256), 0, st, *a);
    if (u <= 4) return launch_pdl("stream_rows", stream_rows_kernel<4>, dim3(rows), dim3(256), 0, st, *a);
    if (u <= 8) return launch_pdl("stream_rows", stream_rows_kernel<8>, dim3(rows), dim3(256), 0, st, *a);
    return launch_pdl("stream_rows", stream_rows_kernel<16>, dim3(rows), dim3(256), 0, st, *a);
}
extern "C" int ckb_launch_row_norm_gate(const float *o, int ldo, const float *w, const float *gate, int ldg, float eps, int n, float mul, void *dst, int ldd, int act, int rows, void *stream)
{
    return launch_pdl("row_norm_gate", row_norm_gate_kernel, dim3(rows), dim3(256), 0, ckb_stream(stream), o, ldo, w, gate, ldg, eps, n, mul, dst, ldd, act);
}

extern "C" int ckb_launch_embed_rows(const int32_t *ids, int rows, int vocab, const void *table, int ld, int n, float scale, float *x, int ldx, void *stream)
{
    return launch_pdl("embed_rows", embed_rows_kernel, dim3(rows), dim3(256), 0, ckb_stream(stream), ids, vocab, static_cast<const __nv_bfloat16 *>(table), ld, n, scale, x, ldx);
}
extern "C" int ckb_launch_rms_rows(const float *src, int lds, const int32_t *idx, int rows, int n, const float *w, float eps, void *dst, int ldd, int width, int act_f32, void *stream)
{
    return launch_pdl("rms_rows", rms_rows_kernel, dim3(rows), dim3(256), 0, ckb_stream(stream), src, lds, idx, n, w, eps, dst, ldd, width, act_f32);
}
extern "C" int ckb_launch_advance_pos(int *pos, int n, void *stream)
{
    return launch_pdl("advance_pos", advance_pos_kernel, dim3(1), dim3(1), 0, ckb_stream(stream), pos, n);
}
extern "C" int ckb_launch_rotate_rows(const RotateRows *a, int n_sets, int rows, int batch, const int *pos, void *stream)
{
    RotateSets sets = {};
    int dims = 0;
    for (int i = 0; i < n_sets && i < 2; ++i) {
        sets.s[i] = a[i];
        if (a[i].dims > dims) dims = a[i].dims;
    }
    return launch_pdl("rotate_rows", rotate_rows_kernel, dim3(rows, n_sets), dim3(256), (size_t)dims * sizeof(float), ckb_stream(stream), sets, batch, pos);
}
extern "C" int ckb_launch_conv_rows(const ConvRows *a, int T, int B, const int *pos, void *stream)
{
    const dim3 grid((T + CONV_TOKENS - 1) / CONV_TOKENS * B, (2 * a->G + a->H + 3) / 4);
    const int n = a->d > a->dv ? a->d : a->dv;
    cudaStream_t st = ckb_stream(stream);
    if (n > 512) return ckb_fail(CKB_ERR_LIMIT, "conv_rows: head size %d", n);
    const int rc = n <= 32 ? launch_pdl("conv_rows", conv_rows_kernel<1>, grid, dim3(128), 0, st, *a, T, B, pos)
                 : n <= 64 ? launch_pdl("conv_rows", conv_rows_kernel<2>, grid, dim3(128), 0, st, *a, T, B, pos)
                 : n <= 128 ? launch_pdl("conv_rows", conv_rows_kernel<4>, grid, dim3(128), 0, st, *a, T, B, pos)
                 : n <= 256 ? launch_pdl("conv_rows", conv_rows_kernel<8>, grid, dim3(128), 0, st, *a, T, B, pos)
                            : launch_pdl("conv_rows", conv_rows_kernel<16>, grid, dim3(128), 0, st, *a, T, B, pos);
    const int channels = 2 * a->G * a->d + a->H * a->dv;
    if (rc || a->taps < 2) return rc;
    return launch_pdl("conv_state", conv_state_kernel, dim3((channels + 127) / 128, B), dim3(128), 0, ckb_stream(stream), *a, T, B, pos);
}
extern "C" int ckb_launch_delta_gates(float *decay, int ldd, const float *a_log, const float *dt_bias, int H, int d, float *beta, int ldb, int rows, void *stream)
{
    return launch_pdl("delta_gates", delta_gates_kernel, dim3(rows), dim3(256), 0, ckb_stream(stream), decay, ldd, a_log, dt_bias, H, d, beta, ldb);
}
extern "C" int ckb_launch_head_norm_gate(const float *o, int ldo, const float *w, int w_stride, const float *gate, int ldg, int gate_kind, float eps, int H, int dv, void *dst, int ldd,
                                         int act, int rows, void *stream)
{
    if (dv % 4 == 0 && dv <= 128 && ldo % 4 == 0 && ldg % 4 == 0 && ldd % 4 == 0 && w_stride % 4 == 0 && (((uintptr_t)o | (uintptr_t)gate | (uintptr_t)w) & 15) == 0 && ((uintptr_t)dst & 15) == 0) {
        const int lanes = dv <= 32 ? 8 : (dv <= 64 ? 16 : 32), heads = 256 / lanes * 4;
        const dim3 grid(rows, (H + heads - 1) / heads);
        cudaStream_t st = ckb_stream(stream);
        if (lanes == 8) return launch_pdl("head_norm_gate", head_norm_gate4_kernel<8>, grid, dim3(256), 0, st, o, ldo, w, w_stride, gate, ldg, gate_kind, eps, H, dv, dst, ldd, act);
        if (lanes == 16) return launch_pdl("head_norm_gate", head_norm_gate4_kernel<16>, grid, dim3(256), 0, st, o, ldo, w, w_stride, gate, ldg, gate_kind, eps, H, dv, dst, ldd, act);
        return launch_pdl("head_norm_gate", head_norm_gate4_kernel<32>, grid, dim3(256), 0, st, o, ldo, w, w_stride, gate, ldg, gate_kind, eps, H, dv, dst, ldd, act);
    }
    return launch_pdl("head_norm_gate", head_norm_gate_kernel, dim3(rows, (H + 3) / 4), dim3(128), 0, ckb_stream(stream), o, ldo, w, w_stride, gate, ldg, gate_kind, eps, H, dv, dst, ldd, act);
}
