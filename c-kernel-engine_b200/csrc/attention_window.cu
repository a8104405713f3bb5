// Softmax attention over a window of cached keys with grouped queries: appending rotated keys, and the fp32 form of the attention itself
// (single tokens, short portions, 32-bit models).  Prompt portions of a bfloat16 cache run in attention_portion.cu.
//
// Attention: a CTA takes up to four query heads of one key head and one row; the CTAs of a cluster share the row's visible keys, a run of
// positions each.  Queries are rotated and normed on the way in, and with one token per sequence the token's own key and value too (they
// go to the cache and are used from shared memory).  A warp takes 4 * KI keys at a time, eight lanes per key, with its own running
// maximum, denominator and sums (base 2); the warps meet in shared memory, then every CTA sends each other one its part of the outputs
// that one finishes (distributed shared memory).
#include <cuda_bf16.h>

#include "device_common.cuh"
#include "launch.h"
#include "mixer_math.cuh"
#include "mixers.h"
#include "pdl.cuh"
#include "runtime.h"

namespace ckb {

constexpr int KV_WARPS = 8, KV_THREADS = KV_WARPS * 32, KV_HEADS = 4, KV_DIM = 256, KV_RANKS = 8;
constexpr float KV_NONE = -1e30f, KV_LOG2E = 1.44269504088896341f;       // KV_NONE: maximum over no key

// sine and cosine of pair i at position p
__device__ __forceinline__ float2 kv_angle(const KvCache &c, float p, int i)
{
    float2 a;
    sincosf(p * c.freq[i], &a.x, &a.y);
    a.x *= c.rot_mul;
    a.y *= c.rot_mul;
    return a;
}

// a vector of n elements as a warp holds it: element lane + 32 i in r[i]
struct KvVector { float r[KV_DIM / 32]; };
__device__ __forceinline__ KvVector kv_fetch(const float *x, int n, int lane)
{
    KvVector v;
#pragma unroll
    for (int i = 0; i < KV_DIM / 32; ++i) v.r[i] = lane + 32 * i < n ? __ldcg(x + lane + 32 * i) : 0.f;
    return v;
}
// rotated (angle(i): sine and cosine of a pair), of unit mean square; swap: KV_DIM floats of the warp's own
template <typename Angle>
__device__ __forceinline__ void kv_turn(const KvCache &c, KvVector &v, int lane, float *swap, Angle angle)
{
    const int half = c.rot_dims / 2;
    __syncwarp();
#pragma unroll
    for (int i = 0; i < KV_DIM / 32; ++i)
        if (lane + 32 * i < 2 * half) swap[lane + 32 * i] = v.r[i];
    __syncwarp();
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < KV_DIM / 32; ++i) {
        const int j = lane + 32 * i;
        if (j < 2 * half) {
            const float other = swap[j < half ? j + half : j - half];
            const float2 a = angle(j < half ? j : j - half);
            v.r[i] = fmaf(v.r[i], a.y, j < half ? -other * a.x : other * a.x);
        }
        ss = fmaf(v.r[i], v.r[i], ss);
    }
    if (!c.unit) return;
    const float rs = 1.f / sqrtf(group_sum<32>(ss) / (float)c.dim + c.eps);
#pragma unroll
    for (int i = 0; i < KV_DIM / 32; ++i) v.r[i] *= rs;
}

__device__ __forceinline__ size_t kv_slot(const KvCache &c, int b, int g, int p) { return ((size_t)b * c.G + g) * c.cap + p % c.cap; }

__global__ __launch_bounds__(KV_THREADS) void kv_append_kernel(const __grid_constant__ KvCache c, const float *q, const float *k, const float *v, int ld, __nv_bfloat16 *q16, int batch,
                                                               const int *pos)
{
    __shared__ float2 turns[KV_DIM / 2];
    __shared__ float swap[KV_WARPS][KV_DIM];
    pdl_wait();
    pdl_trigger();
    const int row = blockIdx.x, b = row % batch, p = __ldcg(pos) + row / batch, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nq = q16 ? c.H : 0, n = nq + c.G;
    auto source = [&](int i) { return i < nq ? q + (size_t)row * ld + i * c.dim : k + (size_t)row * ld + (i - nq) * c.dim; };
    KvVector next = {};
    if (warp < n) next = kv_fetch(source(warp), c.dim, lane);
    if (threadIdx.x < c.rot_dims / 2) turns[threadIdx.x] = kv_angle(c, (float)p, threadIdx.x);
    for (int g = warp; g < c.G; g += KV_WARPS)
        for (int e = lane; e < c.vdim; e += 32) mix_store(c.v, kv_slot(c, b, g, p) * c.vd + e, __ldcg(v + (size_t)row * ld + g * c.vdim + e), c.cache_f32);
    __syncthreads();
    for (int i = warp; i < n; i += KV_WARPS) {
        KvVector x = next;
        if (i + KV_WARPS < n) next = kv_fetch(source(i + KV_WARPS), c.dim, lane);
        kv_turn(c, x, lane, swap[warp], [&](int j) { return turns[j]; });
        if (i < nq) {
            __nv_bfloat16 *d = q16 + ((size_t)row * c.H + i) * c.kd;
#pragma unroll
            for (int e = 0; e < KV_DIM / 32; ++e)
                if (lane + 32 * e < c.kd) d[lane + 32 * e] = __float2bfloat16_rn(x.r[e] * c.scale * KV_LOG2E);
        } else {
            const size_t at = kv_slot(c, b, i - nq, p) * c.kd;
#pragma unroll
            for (int e = 0; e < KV_DIM / 32; ++e)
                if (lane + 32 * e < c.dim) mix_store(c.k, at + lane + 32 * e, x.r[e], c.cache_f32);
        }
    }
}

// N consecutive cached elements as loaded; N a multiple of 2 (bfloat16)
template <bool F32, int N>
struct KvPiece { uint32_t w[F32 ? N : N / 2]; };
template <bool F32, int N>
__device__ __forceinline__ KvPiece<F32, N> kv_load(const void *base, size_t i)
{
    constexpr int WORDS = F32 ? N : N / 2;
    KvPiece<F32, N> r;
    const uint32_t *s = F32 ? static_cast<const uint32_t *>(base) + i : static_cast<const uint32_t *>(base) + i / 2;
    if constexpr (WORDS % 4 == 0) {
#pragma unroll
        for (int j = 0; j < WORDS / 4; ++j) {
            const uint4 x = __ldcg(reinterpret_cast<const uint4 *>(s) + j);
            r.w[4 * j] = x.x; r.w[4 * j + 1] = x.y; r.w[4 * j + 2] = x.z; r.w[4 * j + 3] = x.w;
        }
    } else if constexpr (WORDS == 2) {
        const uint2 x = __ldcg(reinterpret_cast<const uint2 *>(s));
        r.w[0] = x.x; r.w[1] = x.y;
    } else {
        r.w[0] = __ldcg(s);
    }
    return r;
}
template <bool F32, int N>
__device__ __forceinline__ KvPiece<F32, N> kv_pack(const float *s)      // from fp32 values that are numbers of the cache's type
{
    KvPiece<F32, N> r;
#pragma unroll
    for (int j = 0; j < (F32 ? N : N / 2); ++j)
        r.w[j] = F32 ? __float_as_uint(s[j]) : (__float_as_uint(s[(2 * j) % N]) >> 16 | (__float_as_uint(s[(2 * j + 1) % N]) & 0xffff0000u));
    return r;
}
template <bool F32, int N>
__device__ __forceinline__ float kv_get(const KvPiece<F32, N> &p, int i)
{
    if (F32) return __uint_as_float(p.w[i % (F32 ? N : N / 2)]);
    const uint32_t w = p.w[(i / 2) % (F32 ? N : N / 2)];
    return __uint_as_float(i & 1 ? w & 0xffff0000u : w << 16);
}

// store to the same shared-memory variable of CTA `rank` of the cluster
__device__ __forceinline__ void kv_push(float *local, int rank, float v)
{
    uint32_t addr;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(addr) : "r"(smem_u32(local)), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(addr), "f"(v) : "memory");
}
__device__ __forceinline__ void kv_cluster_sync() { asm volatile("barrier.cluster.arrive.aligned;\n\tbarrier.cluster.wait.aligned;" ::: "memory"); }

struct KvAttend {
    KvCache c;
    const float *q, *k, *v;
    int ld;
    void *dst;
    int ldd, act_f32, batch;
};

// PK: 64-element pieces of a key; VE: value elements per lane; KI: keys per lane group and step
template <bool F32, int PK, int VE, int KI>
__global__ __launch_bounds__(KV_THREADS) void kv_attend_kernel(const __grid_constant__ KvAttend a, const int *pos)
{
    constexpr int KEYS = 4 * KI, TILE = KV_WARPS * KEYS, VD = VE * 32;
    __shared__ __align__(16) float qs[KV_HEADS][PK * 64], nk[PK * 64], nv[VD];
    __shared__ float wm[KV_WARPS][KV_HEADS], wl[KV_WARPS][KV_HEADS], rm[KV_RANKS][KV_HEADS], rl[KV_RANKS][KV_HEADS];
    __shared__ __align__(16) float wacc[KV_WARPS][KV_HEADS][VD], racc[KV_HEADS * VD + KV_RANKS], swap[KV_HEADS + 1][PK * 64];       // racc: [sending rank][outputs of this CTA]
    const KvCache &c = a.c;
    const int group = c.H / c.G, blocks = (group + KV_HEADS - 1) / KV_HEADS, g = blockIdx.y / blocks, h0 = g * group + blockIdx.y % blocks * KV_HEADS;
    const int nh = min(KV_HEADS, (g + 1) * group - h0), rank = blockIdx.x, ranks = gridDim.x, row = blockIdx.z, b = row % a.batch;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane >> 3, part = lane & 7;
    for (int i = threadIdx.x; i < KV_HEADS * PK * 64; i += KV_THREADS) (&qs[0][0])[i] = 0.f;
    for (int i = threadIdx.x; i < PK * 64; i += KV_THREADS) nk[i] = 0.f;
    for (int i = threadIdx.x; i < VD; i += KV_THREADS) nv[i] = 0.f;
    if (ranks > 1) kv_cluster_sync();                         // every CTA of the cluster runs: what is sent to it arrives
    pdl_wait();
    pdl_trigger();
    const int p = __ldcg(pos) + row / a.batch, lo = c.window ? max(0, p - c.window + 1) : 0, per = (p - lo + ranks) / ranks;
    const int first = lo + rank * per, end = min(first + per, p + 1), fresh = a.k && end == p + 1 && first < end ? p : -1;       // the key that is not in the cache yet
    const size_t slab = ((size_t)b * c.G + g) * c.cap;
    KvPiece<F32, 8> kr[KI][PK];
    KvPiece<F32, VE> vr[KEYS];
    auto load = [&](int k0) {
#pragma unroll
        for (int i = 0; i < KI; ++i) {
            const int key = k0 + warp * KEYS + i * 4 + sub;
            const size_t at = (slab + key % c.cap) * c.kd;
#pragma unroll
            for (int e = 0; e < PK; ++e) {
                kr[i][e] = {};
                if (key < end && key != fresh && e * 64 + part * 8 < c.kd) kr[i][e] = kv_load<F32, 8>(c.k, at + e * 64 + part * 8);
            }
        }
#pragma unroll
        for (int i = 0; i < KEYS; ++i) {
            const int key = k0 + warp * KEYS + i;
            vr[i] = {};
            if (key < end && key != fresh && lane * VE < c.vd) vr[i] = kv_load<F32, VE>(c.v, (slab + key % c.cap) * c.vd + lane * VE);
        }
    };
    auto angle = [&](int i) { return kv_angle(c, (float)p, i); };
    load(first);
    __syncthreads();                                          // the cleared rows
    if (warp < nh) {
        KvVector x = kv_fetch(a.q + (size_t)row * a.ld + (h0 + warp) * c.dim, c.dim, lane);
        kv_turn(c, x, lane, swap[warp], angle);
#pragma unroll
        for (int e = 0; e < KV_DIM / 32; ++e)
            if (lane + 32 * e < c.dim) qs[warp][lane + 32 * e] = x.r[e] * c.scale * KV_LOG2E;
    } else if (warp == KV_HEADS && fresh >= 0) {
        KvVector x = kv_fetch(a.k + (size_t)row * a.ld + g * c.dim, c.dim, lane);
        kv_turn(c, x, lane, swap[KV_HEADS], angle);
        const size_t at = kv_slot(c, b, g, p) * c.kd;
#pragma unroll
        for (int e = 0; e < KV_DIM / 32; ++e) {
            if (lane + 32 * e >= c.dim) continue;
            nk[lane + 32 * e] = F32 ? x.r[e] : __bfloat162float(__float2bfloat16_rn(x.r[e]));
            if (blockIdx.y % blocks == 0) mix_store(c.k, at + lane + 32 * e, x.r[e], F32);
        }
    } else if (warp == KV_HEADS + 1 && fresh >= 0) {
        const size_t at = kv_slot(c, b, g, p) * c.vd;
        for (int e = lane; e < c.vdim; e += 32) {
            const float x = __ldcg(a.v + (size_t)row * a.ld + g * c.vdim + e);
            nv[e] = F32 ? x : __bfloat162float(__float2bfloat16_rn(x));
            if (blockIdx.y % blocks == 0) mix_store(c.v, at + e, x, F32);
        }
    }
    __syncthreads();
    // a warp's maxima, denominators and sums live in shared memory, so that the loop over the heads stays a loop: little code, which has to
    // come from memory in every step
    if (lane < KV_HEADS) { wm[warp][lane] = KV_NONE; wl[warp][lane] = 0.f; }
    float(*const sums)[VD] = wacc[warp];
    for (int h = 0; h < nh; ++h)
#pragma unroll
        for (int e = 0; e < VE; ++e) sums[h][lane * VE + e] = 0.f;
    for (int k0 = first; k0 < end; k0 += TILE) {
        const int w0 = k0 + warp * KEYS;
        if (fresh >= w0 && fresh < w0 + KEYS) {               // the token's own key and value
#pragma unroll
            for (int i = 0; i < KI; ++i)
                if (w0 + i * 4 + sub == fresh)
#pragma unroll
                    for (int e = 0; e < PK; ++e) kr[i][e] = kv_pack<F32, 8>(nk + e * 64 + part * 8);
#pragma unroll
            for (int i = 0; i < KEYS; ++i)
                if (w0 + i == fresh) vr[i] = kv_pack<F32, VE>(nv + lane * VE);
        }
        __syncwarp();
#pragma unroll 1
        for (int h = 0; h < nh; ++h) {
            float s[KI];
#pragma unroll
            for (int i = 0; i < KI; ++i) s[i] = 0.f;
#pragma unroll
            for (int e = 0; e < PK; ++e) {
                const float4 *qp = reinterpret_cast<const float4 *>(&qs[h][e * 64 + part * 8]);
                const float4 q0 = qp[0], q1 = qp[1];
                const float qv[8] = {q0.x, q0.y, q0.z, q0.w, q1.x, q1.y, q1.z, q1.w};
#pragma unroll
                for (int i = 0; i < KI; ++i)
#pragma unroll
                    for (int j = 0; j < 8; ++j) s[i] = fmaf(qv[j], kv_get<F32, 8>(kr[i][e], j), s[i]);
            }
            const float before = wm[warp][h];
            float mx = before;
#pragma unroll
            for (int i = 0; i < KI; ++i) {
                s[i] = group_sum<8>(s[i]);
                if (w0 + i * 4 + sub >= end) s[i] = -INFINITY;
                mx = fmaxf(mx, s[i]);
            }
            mx = fmaxf(mx, __shfl_xor_sync(~0u, mx, 8));
            mx = fmaxf(mx, __shfl_xor_sync(~0u, mx, 16));
            const float keep = exp2f(before - mx);
            float sum = 0.f, acc[VE];
#pragma unroll
            for (int i = 0; i < KI; ++i) { s[i] = exp2f(s[i] - mx); sum += s[i]; }
            sum += __shfl_xor_sync(~0u, sum, 8);
            sum += __shfl_xor_sync(~0u, sum, 16);
#pragma unroll
            for (int e = 0; e < VE; ++e) acc[e] = sums[h][lane * VE + e] * keep;
#pragma unroll
            for (int i = 0; i < KEYS; ++i) {
                const float w = __shfl_sync(~0u, s[i / 4], (i % 4) * 8);
#pragma unroll
                for (int e = 0; e < VE; ++e) acc[e] = fmaf(w, kv_get<F32, VE>(vr[i], e), acc[e]);
            }
#pragma unroll
            for (int e = 0; e < VE; ++e) sums[h][lane * VE + e] = acc[e];
            __syncwarp();
            if (lane == 0) { wm[warp][h] = mx; wl[warp][h] = fmaf(wl[warp][h], keep, sum); }
        }
        if (k0 + TILE < end) load(k0 + TILE);
    }
    __syncthreads();
    // output i = h * vdim + e of the CTA's heads is finished by rank i / share
    const int outs = nh * c.vdim, share = (outs + ranks - 1) / ranks;
    for (int i = threadIdx.x; i < outs; i += KV_THREADS) {
        const int h = i / c.vdim, e = i % c.vdim;
        float mx = KV_NONE, s = 0.f;
#pragma unroll
        for (int w = 0; w < KV_WARPS; ++w) mx = fmaxf(mx, wm[w][h]);
#pragma unroll
        for (int w = 0; w < KV_WARPS; ++w) s = fmaf(exp2f(wm[w][h] - mx), wacc[w][h][e], s);
        kv_push(&racc[rank * share + i % share], i / share, s);
    }
    if (threadIdx.x < nh * ranks) {
        const int h = threadIdx.x / ranks, to = threadIdx.x % ranks;
        float mx = KV_NONE, d = 0.f;
#pragma unroll
        for (int w = 0; w < KV_WARPS; ++w) mx = fmaxf(mx, wm[w][h]);
#pragma unroll
        for (int w = 0; w < KV_WARPS; ++w) d = fmaf(exp2f(wm[w][h] - mx), wl[w][h], d);
        kv_push(&rm[rank][h], to, mx);
        kv_push(&rl[rank][h], to, d);
    }
    if (ranks > 1) kv_cluster_sync();
    else __syncthreads();
    for (int i = threadIdx.x; i < share && rank * share + i < outs; i += KV_THREADS) {
        const int at = rank * share + i, h = at / c.vdim, e = at % c.vdim;
        float mx = KV_NONE, s = 0.f, d = 0.f;
        for (int r = 0; r < ranks; ++r) mx = fmaxf(mx, rm[r][h]);
        for (int r = 0; r < ranks; ++r) {
            const float f = exp2f(rm[r][h] - mx);
            s = fmaf(f, racc[r * share + i], s);
            d = fmaf(f, rl[r][h], d);
        }
        mix_store(a.dst, (size_t)row * a.ldd + (h0 + h) * c.vdim + e, s / d * c.mul, a.act_f32);
    }
}

template <bool F32, int PK, int VE, int KI>
static int kv_attend_launch(const KvAttend &a, int rows, const int *pos, cudaStream_t st)
{
    const int group = a.c.H / a.c.G, heads = a.c.G * ((group + KV_HEADS - 1) / KV_HEADS);
    // CTAs of a row's keys: a tile each, while there are fewer CTAs than SMs
    const int keys = a.c.window && a.c.window < a.c.cap ? a.c.window : a.c.cap, tile = KV_WARPS * 4 * KI;
    int ranks = (keys + tile - 1) / tile;
    while (ranks > 1 && (ranks > KV_RANKS || (long long)rows * heads * ranks > 2 * ckb_sm_count())) --ranks;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(ranks, heads, rows);
    cfg.blockDim = dim3(KV_THREADS);
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = ranks;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = ckb_tune_get("pdl", 1) ? 2 : 1;
    if (ckb_check_cuda((int)cudaLaunchKernelEx(&cfg, kv_attend_kernel<F32, PK, VE, KI>, a, pos), "kv_attend")) return CKB_ERR_CUDA;
    return ckb_check_launch("kv_attend");
}
template <bool F32, int PK, int KI>
static int kv_attend_pick(const KvAttend &a, int rows, const int *pos, cudaStream_t st)
{
    if (a.c.vd <= 64) return kv_attend_launch<F32, PK, 2, KI>(a, rows, pos, st);
    if (a.c.vd <= 128) return kv_attend_launch<F32, PK, 4, KI>(a, rows, pos, st);
    return kv_attend_launch<F32, PK, 8, (KI > 2 ? 2 : KI)>(a, rows, pos, st);
}

}  // namespace ckb

using namespace ckb;

static int kv_check(const KvCache *c)
{
    if (c->dim > KV_DIM || c->vdim > KV_DIM || c->kd % 8 || c->vd % 8 || c->cap % 64 || c->rot_dims > c->dim || c->H % c->G)
        return ckb_fail(CKB_ERR_LIMIT, "window attention: heads of %d and %d, cache rows of %d and %d, %d slots", c->dim, c->vdim, c->kd, c->vd, c->cap);
    return 0;
}

extern "C" int ckb_launch_kv_append(const KvCache *c, const float *q, const float *k, const float *v, int ld, void *q16, int rows, int batch, const int *pos, void *stream)
{
    if (kv_check(c)) return CKB_ERR_LIMIT;
    return launch_pdl("kv_append", kv_append_kernel, dim3(rows), dim3(KV_THREADS), 0, ckb_stream(stream), *c, q, k, v, ld, static_cast<__nv_bfloat16 *>(q16), batch, pos);
}

extern "C" int ckb_launch_kv_attend(const KvCache *c, const float *q, const float *k, const float *v, int ld, void *dst, int ldd, int act_f32, int rows, int batch, const int *pos, void *stream)
{
    if (kv_check(c)) return CKB_ERR_LIMIT;
    const KvAttend a = {*c, q, k, v, ld, dst, ldd, act_f32, batch};
    cudaStream_t st = ckb_stream(stream);
    if (c->cache_f32) {
        if (c->kd <= 64) return kv_attend_pick<true, 1, 2>(a, rows, pos, st);
        if (c->kd <= 128) return kv_attend_pick<true, 2, 2>(a, rows, pos, st);
        return kv_attend_pick<true, 4, 1>(a, rows, pos, st);
    }
    if (c->kd <= 64) return kv_attend_pick<false, 1, 4>(a, rows, pos, st);
    if (c->kd <= 128) return kv_attend_pick<false, 2, 4>(a, rows, pos, st);
    return kv_attend_pick<false, 4, 2>(a, rows, pos, st);
}
