// Causal attention of a prompt portion on the tensor cores, bfloat16 queries, keys and values, with one of two sources of keys:
//   expanded latents  keys [W_uk c | rotated part] and values W_uv c of every head, for all positions up to the portion's end (the
//                     expansion is one product over the cached latents, ckb_launch_linear_tc)
//   a key/value cache grouped queries, the positions of a window only, slots used in a ring
//
// CTA = 64 queries of one head, four warps of 16.  Keys and values come 64 at a time by cp.async, one tile ahead, into rows whose length
// in 16-byte pieces is odd (ldmatrix without bank conflicts).  Scores are fp32 accumulators of mma.sync.m16n8k16; the online softmax
// runs on them in registers, base 2 (the query carries scale * log2 e); the weights go into the second product as two bfloat16
// pieces (their sum keeps 16 bits), so that it sees fp32-like weights.  Blocks with the most keys start first.
#include <cuda_bf16.h>

#include "act_rows.cuh"
#include "device_common.cuh"
#include "launch.h"
#include "mma_bf16.cuh"
#include "mixers.h"
#include "pdl.cuh"
#include "runtime.h"

namespace ckb {

constexpr int LP_Q = 64, LP_K = 64;

// query rows of a pass -> bfloat16 [rows][H][dim + rot], rotated and scaled
__global__ __launch_bounds__(256) void latent_query_kernel(const __grid_constant__ LatentCache lc, const float *q, int ldq, __nv_bfloat16 *out, float mul, int batch, const int *pos)
{
    extern __shared__ float lq_cs[];
    pdl_wait();
    pdl_trigger();
    const int half = lc.rot / 2, qw = lc.dim + lc.rot;
    const float p = (float)(__ldcg(pos) + (int)blockIdx.x / batch);
    for (int i = threadIdx.x; i < half; i += 256) sincosf(p * lc.freq[i], &lq_cs[half + i], &lq_cs[i]);
    __syncthreads();
    const float *s = q + (size_t)blockIdx.x * ldq;
    __nv_bfloat16 *d = out + (size_t)blockIdx.x * lc.H * qw;
    for (int i = threadIdx.x; i < lc.H * qw; i += 256) {
        const int k = i % qw - lc.dim;
        float v = s[i];
        if (k >= half) v = v * lq_cs[k - half] + s[i - half] * lq_cs[k];
        else if (k >= 0) v = v * lq_cs[k] - s[i + half] * lq_cs[half + k];
        d[i] = __float2bfloat16_rn(v * mul);
    }
}

struct PortionAttention {
    const __nv_bfloat16 *q, *k, *kr, *v;      // q: [T * batch][H][dim + rot]; kr: [positions][rot_ld], the rest of every head's key
    __nv_bfloat16 *out;
    int T, H, group, dim, rot, vdim, rot_ld, ld_out, act, batch, b;      // act: bfloat16, with or without lead rows
    int k_row, v_row;                         // elements between positions (slots)
    size_t k_head, v_head;                    // between key heads; query head h reads key head h / group
    int cap, window;                          // cap: position p lies in slot p % cap (0: in row p); window 0: all positions
    int out_dim;                              // value elements that are stored; the others (up to vdim) are pads
    float mul;
};
constexpr float LP_NONE = -1e30f;             // maximum over no key

template <int DV, bool EXACT>       // vdim <= DV, == DV when EXACT
__global__ __launch_bounds__(128) void portion_attention_kernel(const __grid_constant__ PortionAttention p, const int *pos)
{
    extern __shared__ __align__(16) uint8_t lp_sm[];
    const int qw = p.dim + p.rot, ksteps = (qw + 15) / 16, kld = (ksteps * 2) | 1, vld = (((p.vdim + 15) / 16) * 2) | 1;     // row lengths in 16-byte pieces
    const uint32_t sq = smem_u32(lp_sm), sk = sq + LP_Q * kld * 16, sv = sk + 2 * LP_K * kld * 16;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, t0 = (gridDim.x - 1 - blockIdx.x) * LP_Q;
    const int nq = qw / 8, nd = p.dim / 8, nv = p.vdim / 8;
    // pad columns (an odd number of 8-column pieces, rows past the end) stay zero
    for (int i = threadIdx.x; i < (LP_Q + 2 * LP_K) * kld + 2 * LP_K * vld; i += 128) reinterpret_cast<uint4 *>(lp_sm)[i] = make_uint4(0, 0, 0, 0);
    pdl_wait();
    const int p0 = __ldcg(pos), keys = p0 + min(t0 + LP_Q, p.T), tiles = (keys + LP_K - 1) / LP_K, tile0 = p.window ? max(0, p0 + t0 - p.window + 1) / LP_K : 0;
    const __nv_bfloat16 *kh = p.k + (size_t)(h / p.group) * p.k_head, *vh = p.v + (size_t)(h / p.group) * p.v_head;
    __syncthreads();
    for (int i = threadIdx.x; i < LP_Q * nq; i += 128) {
        const int r = i / nq, c = i % nq;
        if (t0 + r < p.T) lp_cp16(sq + (r * kld + c) * 16, p.q + (((size_t)(t0 + r) * p.batch + p.b) * p.H + h) * qw + c * 8, true);
    }
    auto load = [&](int tile) {
        const int k0 = tile * LP_K, slot0 = p.cap ? k0 % p.cap : k0;          // cap is a multiple of the tile
        const uint32_t dk = sk + (tile & 1) * LP_K * kld * 16, dv = sv + (tile & 1) * LP_K * vld * 16;
        for (int r = warp; r < LP_K; r += 4) {
            const bool in = k0 + r < keys;
            const size_t key = in ? slot0 + r : 0;
            for (int c = lane; c < nq; c += 32)
                lp_cp16(dk + (r * kld + c) * 16, c < nd ? kh + key * p.k_row + c * 8 : p.kr + key * p.rot_ld + (c - nd) * 8, in);
            for (int c = lane; c < nv; c += 32) lp_cp16(dv + (r * vld + c) * 16, vh + key * p.v_row + c * 8, in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(tile0);
    float acc[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    float m[2] = {LP_NONE, LP_NONE}, l[2] = {0.f, 0.f};
    const int mi = lane >> 3, mr = lane & 7;
    const int row = t0 + warp * 16 + (lane >> 2);             // this lane's two query rows: row, row + 8
    const uint32_t qa = sq + ((warp * 16 + (mi & 1) * 8 + mr) * kld + (mi >> 1)) * 16;
    for (int tile = tile0; tile < tiles; ++tile) {
        if (tile + 1 < tiles) {
            load(tile + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t tk = sk + (tile & 1) * LP_K * kld * 16, tv = sv + (tile & 1) * LP_K * vld * 16;
        float s[LP_K / 8][4];
#pragma unroll
        for (int i = 0; i < LP_K / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
        const uint32_t ka = tk + (((mi >> 1) * 8 + mr) * kld + (mi & 1)) * 16;
#pragma unroll 4
        for (int k = 0; k < ksteps; ++k) {
            uint32_t a[4];
            lp_ldsm(a, qa + k * 32);
#pragma unroll
            for (int n = 0; n < LP_K / 16; ++n) {
                uint32_t b[4];
                lp_ldsm(b, ka + n * 16 * kld * 16 + k * 32);
                lp_mma(s[2 * n], a, b[0], b[1]);
                lp_mma(s[2 * n + 1], a, b[2], b[3]);
            }
        }
        if ((tile + 1) * LP_K > p0 + t0 + warp * 16) {        // some key of this tile is past some query of this warp
#pragma unroll
            for (int i = 0; i < LP_K / 8; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (tile * LP_K + i * 8 + (lane & 3) * 2 + (e & 1) > p0 + row + (e >> 1) * 8) s[i][e] = -INFINITY;
        }
        if (p.window && tile * LP_K <= p0 + t0 + warp * 16 + 15 - p.window) {        // some key is before the window of some query
#pragma unroll
            for (int i = 0; i < LP_K / 8; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (tile * LP_K + i * 8 + (lane & 3) * 2 + (e & 1) <= p0 + row + (e >> 1) * 8 - p.window) s[i][e] = -INFINITY;
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float mx = m[r];
#pragma unroll
            for (int i = 0; i < LP_K / 8; ++i) mx = fmaxf(mx, fmaxf(s[i][2 * r], s[i][2 * r + 1]));
            mx = fmaxf(mx, __shfl_xor_sync(~0u, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(~0u, mx, 2));      // finite, also when no key of the tile is visible
            const float keep = exp2f(m[r] - mx);
            m[r] = mx;
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < LP_K / 8; ++i)
#pragma unroll
                for (int e = 2 * r; e < 2 * r + 2; ++e) { s[i][e] = exp2f(s[i][e] - mx); sum += s[i][e]; }
            sum += __shfl_xor_sync(~0u, sum, 1);
            sum += __shfl_xor_sync(~0u, sum, 2);
            l[r] = fmaf(l[r], keep, sum);
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) { acc[i][2 * r] *= keep; acc[i][2 * r + 1] *= keep; }
        }
        const uint32_t va = tv + (((mi & 1) * 8 + mr) * vld + (mi >> 1)) * 16;
#pragma unroll
        for (int k = 0; k < LP_K / 16; ++k) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float x = s[2 * k + (j >> 1)][(j & 1) * 2], y = s[2 * k + (j >> 1)][(j & 1) * 2 + 1];
                lp_split(x, y, hi[j], lo[j]);
            }
#pragma unroll
            for (int n = 0; n < DV / 16; ++n) {
                if (!EXACT && n * 16 >= p.vdim) break;
                uint32_t b[4];
                lp_ldsm_t(b, va + k * 16 * vld * 16 + n * 32);
                lp_mma(acc[2 * n], hi, b[0], b[1]);
                lp_mma(acc[2 * n], lo, b[0], b[1]);
                lp_mma(acc[2 * n + 1], hi, b[2], b[3]);
                lp_mma(acc[2 * n + 1], lo, b[2], b[3]);
            }
        }
        __syncthreads();                                      // before the next load overwrites the other buffer
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        if (row + r * 8 >= p.T) continue;
        const float inv = p.mul / l[r];
        const int at = (row + r * 8) * p.batch + p.b;
        __nv_bfloat16 *o = p.out + act_row(at, p.act) * p.ld_out + h * p.out_dim + (lane & 3) * 2;
        if (act_is_lead(at, p.act)) {
#pragma unroll
            for (int i = 0; i < DV / 8; ++i)
#pragma unroll
                for (int e = 0; e < 2; ++e)
                    if (i * 8 + (lane & 3) * 2 + e < p.out_dim) act_store(p.out, at, p.ld_out, h * p.out_dim + (lane & 3) * 2 + i * 8 + e, acc[i][2 * r + e] * inv, p.act);
        } else if ((p.out_dim & 1) == 0) {
#pragma unroll
            for (int i = 0; i < DV / 8; ++i)
                if (i * 8 + (lane & 3) * 2 < p.out_dim) *reinterpret_cast<__nv_bfloat162 *>(o + i * 8) = __floats2bfloat162_rn(acc[i][2 * r] * inv, acc[i][2 * r + 1] * inv);
        } else {
#pragma unroll
            for (int i = 0; i < DV / 8; ++i)
#pragma unroll
                for (int e = 0; e < 2; ++e)
                    if (i * 8 + (lane & 3) * 2 + e < p.out_dim) o[i * 8 + e] = __float2bfloat16_rn(acc[i][2 * r + e] * inv);
        }
    }
}

static int lp_smem(int qw, int vdim)
{
    const int kld = ((qw + 15) / 16 * 2) | 1, vld = ((vdim + 15) / 16 * 2) | 1;
    return ((LP_Q + 2 * LP_K) * kld + 2 * LP_K * vld) * 16;
}

template <int DV, bool EXACT>
static int lp_launch(const PortionAttention &p, const int *pos, int smem, cudaStream_t st)
{
    static int attr = 48 * 1024;
    if (smem > attr) {
        if (ckb_check_cuda((int)cudaFuncSetAttribute(portion_attention_kernel<DV, EXACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), "portion_attention smem")) return CKB_ERR_CUDA;
        attr = smem;
    }
    return launch_plain("portion_attention", portion_attention_kernel<DV, EXACT>, dim3((p.T + LP_Q - 1) / LP_Q, p.H), dim3(128), (size_t)smem, st, p, pos);
}
template <int DV>
static int lp_exact(const PortionAttention &p, const int *pos, int smem, cudaStream_t st)
{
    return p.vdim == DV ? lp_launch<DV, true>(p, pos, smem, st) : lp_launch<DV, false>(p, pos, smem, st);
}

static int lp_pick(const PortionAttention &p, const int *pos, cudaStream_t st)
{
    const int smem = lp_smem(p.dim + p.rot, p.vdim);
    if (p.vdim <= 64) return lp_exact<64>(p, pos, smem, st);
    if (p.vdim <= 128) return lp_exact<128>(p, pos, smem, st);
    return lp_exact<256>(p, pos, smem, st);
}

}  // namespace ckb

using namespace ckb;

extern "C" int ckb_latent_prefill_takes(const LatentCache *lc)
{
    return !lc->cache_f32 && lc->dim % 8 == 0 && lc->rot % 8 == 0 && lc->vdim % 8 == 0 && lc->vdim <= 256 && lp_smem(lc->dim + lc->rot, lc->vdim) <= 227 * 1024;
}

extern "C" int ckb_launch_latent_query(const LatentCache *lc, const float *q, int ldq, void *out, int rows, int batch, const int *pos, void *stream)
{
    return launch_pdl("latent_query", latent_query_kernel, dim3(rows), dim3(256), (size_t)lc->rot * sizeof(float), ckb_stream(stream), *lc, q, ldq, static_cast<__nv_bfloat16 *>(out),
                      lc->scale * 1.44269504088896341f, batch, pos);
}

extern "C" int ckb_launch_latent_prefill(const LatentCache *lc, const void *q, const void *k, const void *v, void *out, int ld_out, int T, int batch, int b, const int *pos, void *stream)
{
    PortionAttention p = {};
    p.q = static_cast<const __nv_bfloat16 *>(q);
    p.k = static_cast<const __nv_bfloat16 *>(k);
    p.kr = static_cast<const __nv_bfloat16 *>(lc->kr) + (size_t)b * lc->cap * lc->rot_ld;
    p.v = static_cast<const __nv_bfloat16 *>(v);
    p.out = static_cast<__nv_bfloat16 *>(out);
    p.T = T;
    p.H = lc->H;
    p.group = 1;
    p.dim = lc->dim;
    p.rot = lc->rot;
    p.vdim = p.out_dim = lc->vdim;
    p.rot_ld = lc->rot_ld;
    p.ld_out = ld_out;
    p.batch = batch;
    p.b = b;
    p.k_row = lc->H * lc->dim;
    p.v_row = lc->H * lc->vdim;
    p.k_head = lc->dim;
    p.v_head = lc->vdim;
    p.mul = 1.f;
    return lp_pick(p, pos, ckb_stream(stream));
}

extern "C" int ckb_kv_prefill_takes(const KvCache *c) { return !c->cache_f32 && c->vd <= 256 && lp_smem(c->kd, c->vd) <= 227 * 1024; }

extern "C" int ckb_launch_kv_prefill(const KvCache *c, const void *q16, void *dst, int ldd, int act, int T, int batch, const int *pos, void *stream)
{
    PortionAttention p = {};
    p.q = static_cast<const __nv_bfloat16 *>(q16);
    p.out = static_cast<__nv_bfloat16 *>(dst);
    p.T = T;
    p.H = c->H;
    p.group = c->H / c->G;
    p.dim = c->kd;
    p.vdim = c->vd;
    p.out_dim = c->vdim;
    p.ld_out = ldd;
    p.act = act;
    p.batch = batch;
    p.k_row = c->kd;
    p.v_row = c->vd;
    p.k_head = (size_t)c->cap * c->kd;
    p.v_head = (size_t)c->cap * c->vd;
    p.cap = c->cap;
    p.window = c->window;
    p.mul = c->mul;
    for (int b = 0; b < batch; ++b) {
        p.b = b;
        p.k = static_cast<const __nv_bfloat16 *>(c->k) + (size_t)b * c->G * p.k_head;
        p.v = static_cast<const __nv_bfloat16 *>(c->v) + (size_t)b * c->G * p.v_head;
        const int rc = lp_pick(p, pos, ckb_stream(stream));
        if (rc) return rc;
    }
    return 0;
}
