// Latent attention over cached latents: every head's keys and values are linear in the same cached row c, so W_uk is applied to the query
// and W_uv to the weighted sum of latents ("absorbed" form), and the cache is read once for all heads.
//
//   append   norm and rotation of the new rows, stored at their positions
//   absorb   qa = scale * (W_uk[h]^T q | rotated q) per head
//   attend   CTA = (split of the keys, group of 8 heads, row); a warp owns a head: lanes are keys for the scores (32 keys a step, staged
//            in shared memory as fp32) and latent channels for the weighted sum; online softmax in registers, partial results to scratch
//   output   merge of the splits, W_uv, one CTA per (row, head, slice of the head's outputs)
//
// With an fp32 cache all arithmetic is fp32 on the CUDA cores.  With a bfloat16 cache the two products of attend run on the tensor
// cores: 16 heads are the rows of mma.sync.m16n8k16, the query and the weights go in as two bfloat16 pieces each (exact products with
// the cached numbers, fp32 accumulation), softmax stays fp32.
#include <cuda_bf16.h>

#include "device_common.cuh"
#include "launch.h"
#include "mixer_math.cuh"
#include "mixers.h"
#include "mma_bf16.cuh"
#include "pdl.cuh"
#include "runtime.h"

namespace ckb {

constexpr int LA_KEYS = 32, LA_HEADS = 8, LA_PAD = 4, LA_SLICE = 32, LA_ABSORB_COLS = 128;

__device__ __forceinline__ void latent_append_row(const LatentCache &lc, const float *kv, int ldkv, const float *norm_w, float eps, int row, int batch, const int *pos, float *red)
{
    const int p = __ldcg(pos) + row / batch;
    const float *s = kv + (size_t)row * ldkv;
    float ss = 0.f;
    for (int i = threadIdx.x; i < lc.rank; i += 256) { const float v = __ldcg(s + i); ss = fmaf(v, v, ss); }
    ss = group_sum<32>(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += red[i];
    const float rs = 1.f / sqrtf(ss / (float)lc.rank + eps);
    const size_t at = (size_t)(row % batch) * lc.cap + p;
    for (int i = threadIdx.x; i < lc.rank; i += 256) mix_store(lc.c, at * lc.rank_ld + i, __ldcg(s + i) * rs * norm_w[i], lc.cache_f32);
    const int half = lc.rot / 2;
    for (int i = threadIdx.x; i < half; i += 256) {
        float sn, cs;
        sincosf((float)p * lc.freq[i], &sn, &cs);
        const float u = __ldcg(s + lc.rank + i), v = __ldcg(s + lc.rank + half + i);
        mix_store(lc.kr, at * lc.rot_ld + i, u * cs - v * sn, lc.cache_f32);
        mix_store(lc.kr, at * lc.rot_ld + half + i, v * cs + u * sn, lc.cache_f32);
    }
}

__global__ __launch_bounds__(256) void latent_append_kernel(const __grid_constant__ LatentCache lc, const float *kv, int ldkv, const float *norm_w, float eps, int batch, const int *pos)
{
    __shared__ float red[8];
    pdl_wait();
    pdl_trigger();
    latent_append_row(lc, kv, ldkv, norm_w, eps, blockIdx.x, batch, pos, red);
}

struct LatentNew { const float *kv, *norm_w; int ld; float eps; };       // rows to append in the same launch (kv NULL: none)

// grid (column slices of the rank + one block for the rotated part, heads (+ one block per row that appends), rows)
__global__ __launch_bounds__(256) void latent_absorb_kernel(const __grid_constant__ LatentCache lc, const float *q, int ldq, const __nv_bfloat16 *uk, int ld_uk, float *qa,
                                                            const __grid_constant__ LatentNew fresh, int row0, int batch, const int *pos)
{
    extern __shared__ float la_q[];                          // [dim], then [4][LA_ABSORB_COLS] partial sums
    if (blockIdx.y < lc.H && blockIdx.x < gridDim.x - 1)      // weights on their way into L2 meanwhile: 256 bytes a row
        for (int i = threadIdx.x; i < 2 * lc.dim; i += 256) {
            const int col = blockIdx.x * LA_ABSORB_COLS + (i & 1) * 64;
            if (col < ld_uk) asm volatile("prefetch.global.L2 [%0];" ::"l"(uk + (size_t)(blockIdx.y * lc.dim + (i >> 1)) * ld_uk + col));
        }
    pdl_wait();
    pdl_trigger();
    if (blockIdx.y == lc.H) {
        if (blockIdx.x == 0) latent_append_row(lc, fresh.kv, fresh.ld, fresh.norm_w, fresh.eps, row0 + blockIdx.z, batch, pos, la_q);
        return;
    }
    const int h = blockIdx.y, row = row0 + blockIdx.z, qw = lc.dim + lc.rot;
    const float *s = q + (size_t)row * ldq + h * qw;
    float *out = qa + ((size_t)blockIdx.z * lc.H + h) * (lc.rank + lc.rot);
    const int kw = lc.rank_ld + lc.rot_ld;
    __nv_bfloat16 *out2 = reinterpret_cast<__nv_bfloat16 *>(qa) + ((size_t)blockIdx.z * lc.H + h) * 2 * kw;
    auto put = [&](int col, float v) {                       // col < rank: latent, from rank_ld on: rotated part
        if (!lc.q_split) {
            if (col < lc.rank) out[col] = v;
            else if (col >= lc.rank_ld && col - lc.rank_ld < lc.rot) out[lc.rank + col - lc.rank_ld] = v;
            return;
        }
        v *= 1.44269504088896341f;
        const __nv_bfloat16 hi = __float2bfloat16_rn(v);
        out2[col] = hi;
        out2[kw + col] = __float2bfloat16_rn(v - __bfloat162float(hi));
    };
    if (blockIdx.x == gridDim.x - 1) {
        const int half = lc.rot / 2;
        const float p = (float)(__ldcg(pos) + row / batch);
        for (int i = threadIdx.x; i < half; i += 256) {
            float sn, cs;
            sincosf(p * lc.freq[i], &sn, &cs);
            const float u = __ldcg(s + lc.dim + i), v = __ldcg(s + lc.dim + half + i);
            put(lc.rank_ld + i, (u * cs - v * sn) * lc.scale);
            put(lc.rank_ld + half + i, (v * cs + u * sn) * lc.scale);
        }
        for (int i = lc.rot + threadIdx.x; i < lc.rot_ld; i += 256) put(lc.rank_ld + i, 0.f);
        return;
    }
    float *part = la_q + ((lc.dim + 3) & ~3);
    for (int i = threadIdx.x; i < lc.dim; i += 256) la_q[i] = __ldcg(s + i) * lc.scale;
    __syncthreads();
    const int c = blockIdx.x * LA_ABSORB_COLS + (threadIdx.x & 63) * 2, quarter = threadIdx.x >> 6;      // two columns, every fourth row
    float a0 = 0.f, a1 = 0.f;
    if (c < ld_uk) {
        const __nv_bfloat16 *w = uk + (size_t)h * lc.dim * ld_uk + c;
#pragma unroll 16
        for (int i = quarter; i < lc.dim; i += 4) {
            const uint32_t v = *reinterpret_cast<const uint32_t *>(w + (size_t)i * ld_uk);
            a0 = fmaf(__uint_as_float(v << 16), la_q[i], a0);
            a1 = fmaf(__uint_as_float(v & 0xffff0000u), la_q[i], a1);
        }
    }
    part[quarter * LA_ABSORB_COLS + (threadIdx.x & 63) * 2] = a0;
    part[quarter * LA_ABSORB_COLS + (threadIdx.x & 63) * 2 + 1] = a1;
    __syncthreads();
    if (threadIdx.x < LA_ABSORB_COLS) {
        const int col = blockIdx.x * LA_ABSORB_COLS + threadIdx.x;
        // columns of W_uk past the rank are zero
        if (col < lc.rank_ld) put(col, part[threadIdx.x] + part[LA_ABSORB_COLS + threadIdx.x] + part[2 * LA_ABSORB_COLS + threadIdx.x] + part[3 * LA_ABSORB_COLS + threadIdx.x]);
    }
}

// keys of split s: [lo, hi); whole steps of LA_KEYS
__device__ __forceinline__ void latent_range(int keys, int splits, int s, int &lo, int &hi)
{
    const int steps = (keys + LA_KEYS - 1) / LA_KEYS, per = (steps + splits - 1) / splits * LA_KEYS;
    lo = min(s * per, keys);
    hi = min(lo + per, keys);
}

template <int NC>       // latent channels per lane: rank <= 32 * NC
__global__ __launch_bounds__(256) void latent_attend_kernel(const __grid_constant__ LatentCache lc, const float *qa, float *part, int splits, int row0, int batch, const int *pos)
{
    extern __shared__ __align__(16) float la_sm[];
    const int width = (lc.rank + lc.rot + 3) & ~3, ld = width + LA_PAD;
    float *kt = la_sm, *qs = kt + LA_KEYS * ld, *ps = qs + LA_HEADS * width;       // keys, queries, probabilities [8][32]
    pdl_wait();
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = row0 + blockIdx.z, b = row % batch;
    const int h = blockIdx.y * LA_HEADS + warp, keys = __ldcg(pos) + row / batch + 1;
    int lo, hi;
    latent_range(keys, splits, blockIdx.x, lo, hi);
    const int heads = min(LA_HEADS, lc.H - (int)blockIdx.y * LA_HEADS);
    for (int i = threadIdx.x; i < LA_HEADS * width; i += 256) {
        const int hh = i / width, k = i % width;
        qs[i] = hh < heads && k < lc.rank + lc.rot ? __ldcg(qa + ((size_t)blockIdx.z * lc.H + blockIdx.y * LA_HEADS + hh) * (lc.rank + lc.rot) + k) : 0.f;
    }
    float m = -INFINITY, l = 0.f, acc[NC];
#pragma unroll
    for (int i = 0; i < NC; ++i) acc[i] = 0.f;
    for (int k0 = lo; k0 < hi; k0 += LA_KEYS) {
        __syncthreads();
        const int n = min(LA_KEYS, hi - k0);
        const size_t at = (size_t)b * lc.cap + k0;
        for (int key = warp; key < LA_KEYS; key += 8) {       // a warp per key row; rows past the end are zero
            float *dst = kt + key * ld;
            if (lc.cache_f32) {
                const float *c = static_cast<const float *>(lc.c) + (at + key) * lc.rank_ld, *r = static_cast<const float *>(lc.kr) + (at + key) * lc.rot_ld;
                for (int i = lane; i < width; i += 32) dst[i] = key >= n || i >= lc.rank + lc.rot ? 0.f : (i < lc.rank ? __ldcg(c + i) : __ldcg(r + i - lc.rank));
            } else {
                const __nv_bfloat16 *c = static_cast<const __nv_bfloat16 *>(lc.c) + (at + key) * lc.rank_ld, *r = static_cast<const __nv_bfloat16 *>(lc.kr) + (at + key) * lc.rot_ld;
                for (int i = lane; i < width; i += 32)
                    dst[i] = key >= n || i >= lc.rank + lc.rot ? 0.f : __bfloat162float(i < lc.rank ? c[i] : r[i - lc.rank]);
            }
        }
        __syncthreads();
        if (warp < heads) {
            float s = 0.f;
            const float4 *kp = reinterpret_cast<const float4 *>(kt + lane * ld), *qp = reinterpret_cast<const float4 *>(qs + warp * width);
#pragma unroll 4
            for (int i = 0; i < width / 4; ++i) {
                const float4 a = kp[i], q = qp[i];
                s = fmaf(a.x, q.x, fmaf(a.y, q.y, fmaf(a.z, q.z, fmaf(a.w, q.w, s))));
            }
            if (lane >= n) s = -INFINITY;
            float mx = s;
#pragma unroll
            for (int o = 16; o; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(~0u, mx, o));
            mx = fmaxf(mx, m);                                // finite: every step has a visible key
            const float p = expf(s - mx), keep = expf(m - mx);
            m = mx;
            l = fmaf(l, keep, group_sum<32>(p));
            ps[warp * 32 + lane] = p;
            __syncwarp();
#pragma unroll
            for (int i = 0; i < NC; ++i) acc[i] *= keep;
            for (int key = 0; key < n; ++key) {
                const float w = ps[warp * 32 + key];
#pragma unroll
                for (int i = 0; i < NC; ++i) acc[i] = fmaf(w, kt[key * ld + min(lane + 32 * i, width - 1)], acc[i]);
            }
            __syncwarp();
        }
    }
    if (warp >= heads) return;
    float *dst = part + (((size_t)blockIdx.z * lc.H + h) * splits + blockIdx.x) * (lc.rank + 2);
#pragma unroll
    for (int i = 0; i < NC; ++i)
        if (lane + 32 * i < lc.rank) dst[lane + 32 * i] = acc[i];
    if (lane == 0) { dst[lc.rank] = m; dst[lc.rank + 1] = l; }
}

constexpr int LM_KEYS = 64, LM_HEADS = 16;

// grid (splits, groups of 16 heads, rows), eight warps: in the scores a warp owns 8 keys, in the weighted sum every eighth group of 16 latents
template <int NG>       // groups of 16 latents per warp: rank_ld <= 128 * NG
__global__ __launch_bounds__(256) void latent_attend_mma_kernel(const __grid_constant__ LatentCache lc, const float *qa, float *part, int splits, int row0, int batch, const int *pos)
{
    extern __shared__ __align__(16) uint8_t lm_sm[];
    const int kw = lc.rank_ld + lc.rot_ld, ld = kw / 8 | 1;   // row length in 16-byte pieces, odd: ldmatrix without bank conflicts
    const uint32_t kt = smem_u32(lm_sm), qh = kt + LM_KEYS * ld * 16, ql = qh + LM_HEADS * ld * 16;
    __shared__ __align__(16) float sc[LM_HEADS][LM_KEYS + 4];
    __shared__ __align__(16) __nv_bfloat16 pr[2][LM_HEADS][LM_KEYS + 8];      // the weights' two pieces
    __shared__ float keep[LM_HEADS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = row0 + blockIdx.z, b = row % batch;
    const int h0 = blockIdx.y * LM_HEADS, heads = min(LM_HEADS, lc.H - h0), mi = lane >> 3, mr = lane & 7;
    pdl_wait();
    pdl_trigger();
    const int keys = __ldcg(pos) + row / batch + 1, tiles = (keys + LM_KEYS - 1) / LM_KEYS, per = (tiles + splits - 1) / splits;
    const int first = min((int)blockIdx.x * per, tiles), last = min(first + per, tiles);
    const __nv_bfloat16 *c = static_cast<const __nv_bfloat16 *>(lc.c) + (size_t)b * lc.cap * lc.rank_ld, *kr = static_cast<const __nv_bfloat16 *>(lc.kr) + (size_t)b * lc.cap * lc.rot_ld;
    const int nc = lc.rank_ld / 8, nk = kw / 8;
    auto load = [&](int tile) {
        for (int r = warp; r < LM_KEYS; r += 8) {
            const bool in = tile * LM_KEYS + r < keys;
            const size_t key = in ? tile * LM_KEYS + r : 0;
            for (int i = lane; i < nk; i += 32) lp_cp16(kt + (r * ld + i) * 16, i < nc ? c + key * lc.rank_ld + i * 8 : kr + key * lc.rot_ld + (i - nc) * 8, in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const __nv_bfloat16 *q2 = reinterpret_cast<const __nv_bfloat16 *>(qa) + ((size_t)blockIdx.z * lc.H + h0) * 2 * kw;
    for (int r = warp; r < 2 * LM_HEADS; r += 8)              // row 2 h + piece
        for (int i = lane; i < nk; i += 32) lp_cp16(((r & 1) ? ql : qh) + ((r >> 1) * ld + i) * 16, q2 + (size_t)((r >> 1) < heads ? r : 0) * kw + i * 8, (r >> 1) < heads);
    if (first < last) load(first);
    float acc[NG][2][4];
#pragma unroll
    for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[g][0][e] = acc[g][1][e] = 0.f;
    float m = -INFINITY, l = 0.f;                             // of head threadIdx.x / 16, in its 16 lanes
    const uint32_t a_off = (((mi & 1) * 8 + mr) * ld + (mi >> 1)) * 16, kb = kt + ((warp * 8 + mr) * ld + mi) * 16;
    for (int tile = first; tile < last; ++tile) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 2
        for (int k = 0; k < kw / 16; k += 2) {
            uint32_t bk[4], hi[4], lo[4];
            lp_ldsm(bk, kb + k * 32);                         // 8 keys x 32 columns
            lp_ldsm(hi, qh + a_off + k * 32);
            lp_ldsm(lo, ql + a_off + k * 32);
            lp_mma(s, hi, bk[0], bk[1]);
            lp_mma(s, lo, bk[0], bk[1]);
            lp_ldsm(hi, qh + a_off + k * 32 + 32);
            lp_ldsm(lo, ql + a_off + k * 32 + 32);
            lp_mma(s, hi, bk[2], bk[3]);
            lp_mma(s, lo, bk[2], bk[3]);
        }
        *reinterpret_cast<float2 *>(&sc[lane >> 2][warp * 8 + (lane & 3) * 2]) = make_float2(s[0], s[1]);
        *reinterpret_cast<float2 *>(&sc[(lane >> 2) + 8][warp * 8 + (lane & 3) * 2]) = make_float2(s[2], s[3]);
        __syncthreads();
        {
            const int h = threadIdx.x >> 4, k0 = (threadIdx.x & 15) * 4;
            float x[4], mx = m, sum = 0.f;
            const float4 v = *reinterpret_cast<const float4 *>(&sc[h][k0]);
            x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                if (tile * LM_KEYS + k0 + i >= keys) x[i] = -INFINITY;
                mx = fmaxf(mx, x[i]);
            }
#pragma unroll
            for (int o = 8; o; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(~0u, mx, o));         // finite: every tile has a visible key
#pragma unroll
            for (int i = 0; i < 4; ++i) { x[i] = exp2f(x[i] - mx); sum += x[i]; }
            const float f = exp2f(m - mx);
            m = mx;
            l = fmaf(l, f, group_sum<16>(sum));
            if ((threadIdx.x & 15) == 0) keep[h] = f;
            uint2 hi, lo;
            lp_split(x[0], x[1], hi.x, lo.x);
            lp_split(x[2], x[3], hi.y, lo.y);
            *reinterpret_cast<uint2 *>(&pr[0][h][k0]) = hi;
            *reinterpret_cast<uint2 *>(&pr[1][h][k0]) = lo;
        }
        __syncthreads();
        const float f0 = keep[lane >> 2], f1 = keep[(lane >> 2) + 8];
#pragma unroll
        for (int g = 0; g < NG; ++g)
#pragma unroll
            for (int n = 0; n < 2; ++n) { acc[g][n][0] *= f0; acc[g][n][1] *= f0; acc[g][n][2] *= f1; acc[g][n][3] *= f1; }
#pragma unroll
        for (int k = 0; k < LM_KEYS / 16; ++k) {
            uint32_t hi[4], lo[4];
            lp_ldsm(hi, smem_u32(&pr[0][(mi & 1) * 8 + mr][k * 16 + (mi >> 1) * 8]));
            lp_ldsm(lo, smem_u32(&pr[1][(mi & 1) * 8 + mr][k * 16 + (mi >> 1) * 8]));
#pragma unroll
            for (int g = 0; g < NG; ++g) {
                const int col = (g * 8 + warp) * 16;
                if (col >= lc.rank_ld) break;
                uint32_t bv[4];
                lp_ldsm_t(bv, kt + ((k * 16 + (mi & 1) * 8 + mr) * ld + col / 8 + (mi >> 1)) * 16);
                lp_mma(acc[g][0], hi, bv[0], bv[1]);
                lp_mma(acc[g][0], lo, bv[0], bv[1]);
                lp_mma(acc[g][1], hi, bv[2], bv[3]);
                lp_mma(acc[g][1], lo, bv[2], bv[3]);
            }
        }
        __syncthreads();                                      // the tile is read: the next one may overwrite it
        if (tile + 1 < last) load(tile + 1);
    }
    float *dst = part + (((size_t)blockIdx.z * lc.H + h0) * splits + blockIdx.x) * (lc.rank + 2);
    const size_t hs = (size_t)splits * (lc.rank + 2);
#pragma unroll
    for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int h = (lane >> 2) + (e >> 1) * 8, col = (g * 8 + warp) * 16 + n * 8 + (lane & 3) * 2 + (e & 1);
                if (first < last && h < heads && col < lc.rank) dst[h * hs + col] = acc[g][n][e];
            }
    const int h = threadIdx.x >> 4;
    if ((threadIdx.x & 15) == 0 && h < heads) {
        dst[h * hs + lc.rank] = m * 0.693147180559945309f;    // natural logarithm, as the fp32 kernel leaves it
        dst[h * hs + lc.rank + 1] = l;
    }
}

__global__ __launch_bounds__(256) void latent_output_kernel(const __grid_constant__ LatentCache lc, const float *part, int splits, const __nv_bfloat16 *uv, int ld_uv, void *dst, int ldd,
                                                            int act_f32, int row0, int batch, const int *pos)
{
    extern __shared__ float lo_sm[];                         // [ld_uv] merged latent, [splits] weights
    float *lat = lo_sm, *wt = lo_sm + ld_uv;
    const int h = blockIdx.y, row = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float *src = part + ((size_t)row * lc.H + h) * splits * (lc.rank + 2);
    for (int i = threadIdx.x; i < LA_SLICE * ld_uv / 64; i += 256) {          // weights on their way into L2 meanwhile
        const int r = blockIdx.x * LA_SLICE + i / (ld_uv / 64);
        if (r < lc.vdim) asm volatile("prefetch.global.L2 [%0];" ::"l"(uv + (size_t)(h * lc.vdim + r) * ld_uv + i % (ld_uv / 64) * 64));
    }
    pdl_wait();
    pdl_trigger();
    const int step = lc.q_split ? LM_KEYS : LA_KEYS, steps = (__ldcg(pos) + (row0 + row) / batch + step) / step, used = (steps + (steps + splits - 1) / splits - 1) / ((steps + splits - 1) / splits);
    if (warp == 0) {                                          // splits from `used` on had no keys
        float m = -INFINITY;
        for (int s = lane; s < used; s += 32) m = fmaxf(m, __ldcg(src + (size_t)s * (lc.rank + 2) + lc.rank));
#pragma unroll
        for (int o = 16; o; o >>= 1) m = fmaxf(m, __shfl_xor_sync(~0u, m, o));
        float l = 0.f;
        for (int s = lane; s < used; s += 32) {
            const float w = expf(__ldcg(src + (size_t)s * (lc.rank + 2) + lc.rank) - m);
            wt[s] = w;
            l = fmaf(w, __ldcg(src + (size_t)s * (lc.rank + 2) + lc.rank + 1), l);
        }
        l = group_sum<32>(l);
        for (int s = lane; s < used; s += 32) wt[s] /= l;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < ld_uv; i += 256) {
        float v = 0.f;
        if (i < lc.rank)
#pragma unroll 16
            for (int s = 0; s < used; ++s) v = fmaf(wt[s], __ldcg(src + (size_t)s * (lc.rank + 2) + i), v);
        lat[i] = v;
    }
    __syncthreads();
    const int i0 = blockIdx.x * LA_SLICE + warp;              // four rows per warp
    float v[LA_SLICE / 8] = {};
    for (int k = lane * 8; k < ld_uv; k += 256) {
        uint4 w[LA_SLICE / 8];
#pragma unroll
        for (int r = 0; r < LA_SLICE / 8; ++r)
            w[r] = i0 + r * 8 < lc.vdim ? *reinterpret_cast<const uint4 *>(uv + (size_t)(h * lc.vdim + i0 + r * 8) * ld_uv + k) : make_uint4(0, 0, 0, 0);
#pragma unroll
        for (int r = 0; r < LA_SLICE / 8; ++r) {
            const uint32_t x[4] = {w[r].x, w[r].y, w[r].z, w[r].w};
#pragma unroll
            for (int e = 0; e < 4; ++e) v[r] = fmaf(__uint_as_float(x[e] << 16), lat[k + 2 * e], fmaf(__uint_as_float(x[e] & 0xffff0000u), lat[k + 2 * e + 1], v[r]));
        }
    }
#pragma unroll
    for (int r = 0; r < LA_SLICE / 8; ++r) {
        v[r] = group_sum<32>(v[r]);
        if (lane == 0 && i0 + r * 8 < lc.vdim) mix_store(dst, (size_t)row * ldd + h * lc.vdim + i0 + r * 8, v[r], act_f32);
    }
}

static int lm_smem(const LatentCache *lc) { return (LM_KEYS + 2 * LM_HEADS) * (((lc->rank_ld + lc->rot_ld) / 8) | 1) * 16; }

template <int NG>
static int la_attend_mma(const LatentCache *lc, const float *qa, float *part, int splits, int rows, int row0, int batch, const int *pos, int smem, cudaStream_t st)
{
    static int attr = 0;
    if (smem > attr) {
        if (ckb_check_cuda((int)cudaFuncSetAttribute(latent_attend_mma_kernel<NG>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), "latent_attend_mma smem")) return CKB_ERR_CUDA;
        attr = smem;
    }
    return launch_pdl("latent_attend_mma", latent_attend_mma_kernel<NG>, dim3(splits, (lc->H + LM_HEADS - 1) / LM_HEADS, rows), dim3(256), (size_t)smem, st, *lc, qa, part, splits, row0, batch, pos);
}

template <int NC>
static int la_attend(const LatentCache *lc, const float *qa, float *part, int splits, int rows, int row0, int batch, const int *pos, cudaStream_t st)
{
    const int width = (lc->rank + lc->rot + 3) & ~3;
    const int smem = (LA_KEYS * (width + LA_PAD) + LA_HEADS * width + LA_HEADS * 32) * (int)sizeof(float);
    static int attr = 48 * 1024;
    if (smem > 227 * 1024) return ckb_fail(CKB_ERR_LIMIT, "latent attention: rows of %d elements do not fit into shared memory", width);
    if (smem > attr) {
        if (ckb_check_cuda((int)cudaFuncSetAttribute(latent_attend_kernel<NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), "latent_attend smem")) return CKB_ERR_CUDA;
        attr = smem;
    }
    return launch_pdl("latent_attend", latent_attend_kernel<NC>, dim3(splits, (lc->H + LA_HEADS - 1) / LA_HEADS, rows), dim3(256), (size_t)smem, st, *lc, qa, part, splits, row0, batch, pos);
}

}  // namespace ckb

using namespace ckb;

extern "C" int ckb_latent_q_split(const LatentCache *lc)
{
    return !lc->cache_f32 && lc->rank_ld % 32 == 0 && lc->rot_ld % 32 == 0 && lc->rank_ld <= 1024 && lm_smem(lc) <= 210 * 1024 && ckb_tune_get("latent_mma", 1);
}
extern "C" int ckb_launch_latent_append(const LatentCache *lc, const float *kv, int ldkv, const float *norm_w, float eps, int rows, int batch, const int *pos, void *stream)
{
    return launch_pdl("latent_append", latent_append_kernel, dim3(rows), dim3(256), 0, ckb_stream(stream), *lc, kv, ldkv, norm_w, eps, batch, pos);
}
static int la_absorb(const LatentCache *lc, const float *q, int ldq, const void *uk, int ld_uk, float *qa, const LatentNew &fresh, int rows, int row0, int batch, const int *pos, void *stream)
{
    const size_t smem = (((size_t)lc->dim + 3) / 4 * 4 + 4 * LA_ABSORB_COLS) * sizeof(float);
    return launch_pdl("latent_absorb", latent_absorb_kernel, dim3((lc->rank + LA_ABSORB_COLS - 1) / LA_ABSORB_COLS + 1, lc->H + (fresh.kv ? 1 : 0), rows), dim3(256), smem, ckb_stream(stream),
                      *lc, q, ldq, static_cast<const __nv_bfloat16 *>(uk), ld_uk, qa, fresh, row0, batch, pos);
}
extern "C" int ckb_launch_latent_absorb(const LatentCache *lc, const float *q, int ldq, const void *uk, int ld_uk, float *qa, int rows, int row0, int batch, const int *pos, void *stream)
{
    return la_absorb(lc, q, ldq, uk, ld_uk, qa, LatentNew{nullptr, nullptr, 0, 0.f}, rows, row0, batch, pos, stream);
}
extern "C" int ckb_launch_latent_absorb_append(const LatentCache *lc, const float *q, int ldq, const void *uk, int ld_uk, float *qa, const float *kv, int ldkv, const float *norm_w, float eps,
                                               int rows, int batch, const int *pos, void *stream)
{
    return la_absorb(lc, q, ldq, uk, ld_uk, qa, LatentNew{kv, norm_w, ldkv, eps}, rows, 0, batch, pos, stream);
}
extern "C" int ckb_launch_latent_attend(const LatentCache *lc, const float *qa, float *part, int splits, int rows, int row0, int batch, const int *pos, void *stream)
{
    cudaStream_t st = ckb_stream(stream);
    if (lc->q_split) {
        const int mma_smem = lm_smem(lc);
        if (lc->rank_ld <= 128) return la_attend_mma<1>(lc, qa, part, splits, rows, row0, batch, pos, mma_smem, st);
        if (lc->rank_ld <= 256) return la_attend_mma<2>(lc, qa, part, splits, rows, row0, batch, pos, mma_smem, st);
        if (lc->rank_ld <= 512) return la_attend_mma<4>(lc, qa, part, splits, rows, row0, batch, pos, mma_smem, st);
        return la_attend_mma<8>(lc, qa, part, splits, rows, row0, batch, pos, mma_smem, st);
    }
    if (lc->rank <= 128) return la_attend<4>(lc, qa, part, splits, rows, row0, batch, pos, st);
    if (lc->rank <= 256) return la_attend<8>(lc, qa, part, splits, rows, row0, batch, pos, st);
    if (lc->rank <= 512) return la_attend<16>(lc, qa, part, splits, rows, row0, batch, pos, st);
    if (lc->rank <= 1024) return la_attend<32>(lc, qa, part, splits, rows, row0, batch, pos, st);
    return ckb_fail(CKB_ERR_LIMIT, "latent attention: kv_rank %d (at most 1024)", lc->rank);
}
extern "C" int ckb_launch_latent_output(const LatentCache *lc, const float *part, int splits, const void *uv, int ld_uv, void *dst, int ldd, int act_f32, int rows, int row0, int batch,
                                        const int *pos, void *stream)
{
    const size_t smem = ((size_t)ld_uv + splits) * sizeof(float);
    return launch_pdl("latent_output", latent_output_kernel, dim3((lc->vdim + LA_SLICE - 1) / LA_SLICE, lc->H, rows), dim3(256), smem, ckb_stream(stream), *lc, part, splits,
                      static_cast<const __nv_bfloat16 *>(uv), ld_uv, dst, ldd, act_f32, row0, batch, pos);
}
