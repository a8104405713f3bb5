// One token per sequence through a recurrent mixer, in one launch between the two products of its layer.
//
// The CTAs of a cluster share a head: each takes 32 columns of its state (four per warp, rows spread over the lanes as in
// mixer_recurrence.cu).  Retention: rotation of q and k, S = a S + k v^T, o = S^T q.  Delta rule: convolution with SiLU and unit length,
// the head's decays and output gates from their low-rank inputs (each CTA computes a share of the decays and writes it into the
// others' shared memory), the gated update.  Wkv: decays from their low-rank input in the same way, read-out with the bonus before the
// update.  Lightning: S = a S + k v^T, o = S^T q, its norm left to the output product.  The head norm needs the sum of squares over all
// columns: partial sums are exchanged the same way.  The state is fetched before the dependency wait of the programmatic launch: whatever wrote it last finished at least two
// launches ago.
#include <cuda_bf16.h>

#include "device_common.cuh"
#include "launch.h"
#include "mixer_lanes.cuh"
#include "mixer_math.cuh"
#include "mixers.h"
#include "pdl.cuh"
#include "runtime.h"

namespace ckb {

constexpr int RS_COLS = 32, RS_WARPS = RS_COLS / 4, RS_THREADS = RS_WARPS * 32;

__device__ __forceinline__ void rs_cluster_sync() { asm volatile("barrier.cluster.arrive.aligned;\n\tbarrier.cluster.wait.aligned;" ::: "memory"); }
// store to the same shared-memory variable of CTA `rank` of the cluster
__device__ __forceinline__ void rs_store_remote(float *local, int rank, float v)
{
    uint32_t addr;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(addr) : "r"(smem_u32(local)), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(addr), "f"(v) : "memory");
}
// dots of up to four bfloat16 rows (first, first + step, ..; n elements, a multiple of 64) with fp32 values, one warp; rows from `rows` on
// are left out
__device__ __forceinline__ void rs_dot4(float (&v)[4], const __nv_bfloat16 *w, int first, int step, int rows, const float *x, int n, int lane)
{
    v[0] = v[1] = v[2] = v[3] = 0.f;
#pragma unroll 2
    for (int k = lane; k < n / 2; k += 32) {
        uint32_t u[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) u[r] = first + r * step < rows ? reinterpret_cast<const uint32_t *>(w + (size_t)(first + r * step) * n)[k] : 0u;
        const float x0 = x[2 * k], x1 = x[2 * k + 1];
#pragma unroll
        for (int r = 0; r < 4; ++r) v[r] = fmaf(__uint_as_float(u[r] << 16), x0, fmaf(__uint_as_float(u[r] & 0xffff0000u), x1, v[r]));
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) v[r] = group_sum<32>(v[r]);
}

template <int RPL, int KIND>
__global__ __launch_bounds__(RS_THREADS) void recur_step_kernel(const __grid_constant__ RecurStep a, int B, const int *pos)
{
    constexpr bool DELTA = KIND == STEP_DELTA, WKV = KIND == STEP_WKV, LIGHTNING = KIND == STEP_LIGHTNING, LOW = DELTA || WKV;
    constexpr int DP = RPL * 32;
    extern __shared__ float rs_low[];                        // low-rank inputs of decay and gate
    __shared__ __align__(16) float q[DP], k[DP], g[DP];
    __shared__ float v[RS_COLS], gate[RS_COLS], o[RS_COLS], part[8], red[2][RS_WARPS];
    const RecurRows &r = a.r;
    const int rank = blockIdx.x, ranks = gridDim.x, h = blockIdx.y, b = blockIdx.z, kh = h / (r.H / r.G);
    const int col0 = rank * RS_COLS, ncol = min(RS_COLS, r.dv - col0), warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wcol = warp * 4;
    float *st = r.state + (((size_t)b * r.H + h) * r.dv + col0 + wcol) * DP + lane * RPL;
    float S[4][RPL];
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        RecVec<RPL> x = {};
        if (wcol + c < ncol) x = rec_read<RPL>(st + (size_t)c * DP);
#pragma unroll
        for (int i = 0; i < RPL; ++i) S[c][i] = x.v[i];
    }
    if (LOW) {                                                // weights of the low-rank products on their way into L2 meanwhile
        const int share = (r.d + ranks - 1) / ranks, n1 = max(0, min((rank + 1) * share, r.d) - rank * share) * a.ld_a2 / 64, n2 = DELTA ? ncol * a.ld_g2 / 64 : 0;
        const char *w1 = reinterpret_cast<const char *>(static_cast<const __nv_bfloat16 *>(a.a2) + (size_t)(h * r.d + rank * share) * a.ld_a2);
        const char *w2 = reinterpret_cast<const char *>(static_cast<const __nv_bfloat16 *>(a.g2) + (size_t)(h * r.dv + col0) * a.ld_g2);
        for (int i = threadIdx.x; i < n1 + n2; i += RS_THREADS) asm volatile("prefetch.global.L2 [%0];" ::"l"(i < n1 ? w1 + (size_t)i * 128 : w2 + (size_t)(i - n1) * 128));
    }
    for (int i = threadIdx.x; i < DP; i += RS_THREADS) { q[i] = k[i] = 0.f; g[i] = 1.f; }
    if (threadIdx.x < RS_COLS) v[threadIdx.x] = gate[threadIdx.x] = 0.f;
    if (threadIdx.x < 8) part[threadIdx.x] = 0.f;
    __syncthreads();
    rs_cluster_sync();                                        // every CTA of the cluster runs and has cleared its exchange buffers
    if (!LIGHTNING || !a.ready) pdl_wait();
    pdl_trigger();
    const int p = KIND == STEP_RETENTION || DELTA ? __ldcg(pos) : 0;
    const float *qz = r.q + (size_t)b * r.ldq + kh * r.d, *kz = r.k + (size_t)b * r.ldk + kh * r.d, *vz = r.v + (size_t)b * r.ldv + h * r.dv + col0;
    float beta = 0.f, qmul = 1.f, kmul = 1.f;
    if (DELTA) {
        const int channels = 2 * r.G * r.d + r.H * r.dv;
        float *ring = a.conv_state + (size_t)b * a.taps * channels;
        const int now = p % a.taps;
        // channels of this head's q and k, then this CTA's columns of v
        float sq = 0.f, sk = 0.f;
        for (int i = threadIdx.x; i < 2 * r.d + ncol; i += RS_THREADS) {
            const int kind = i < r.d ? 0 : (i < 2 * r.d ? 1 : 2), j = i - kind * r.d;
            const int ch = kind == 0 ? kh * r.d + j : (kind == 1 ? (r.G + kh) * r.d + j : 2 * r.G * r.d + h * r.dv + col0 + j);
            const float x = __ldcg((kind == 0 ? qz : (kind == 1 ? kz : vz)) + j), *w = a.conv_w + (size_t)ch * a.taps;
            float acc = x * w[a.taps - 1];
#pragma unroll 4
            for (int t = 1; t < a.taps; ++t) {
                const int slot = now - t + (now < t ? a.taps : 0);
                const float past = __ldcg(ring + (size_t)slot * channels + ch);
                acc = fmaf(w[a.taps - 1 - t], p >= t ? past : 0.f, acc);
            }
            acc = mix_silu(acc);
            // nobody reads slot `now` in this step; heads that share a q/k head all see the same input, one of them stores it
            if (kind == 2 || (rank == 0 && h % (r.H / r.G) == 0)) ring[(size_t)now * channels + ch] = x;
            if (kind == 0) { q[j] = acc; sq = fmaf(acc, acc, sq); }
            else if (kind == 1) { k[j] = acc; sk = fmaf(acc, acc, sk); }
            else v[j] = acc;
        }
        sq = group_sum<32>(sq);
        sk = group_sum<32>(sk);
        if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
        float *gl = rs_low + a.ld_a2;
        for (int i = threadIdx.x; i < a.ld_a2; i += RS_THREADS) rs_low[i] = __ldcg(a.a_low + (size_t)b * a.ld_low + i);
        for (int i = threadIdx.x; i < a.ld_g2; i += RS_THREADS) gl[i] = __ldcg(a.g_low + (size_t)b * a.ld_low + i);
        __syncthreads();
        sq = sk = 0.f;
#pragma unroll
        for (int i = 0; i < RS_WARPS; ++i) { sq += red[0][i]; sk += red[1][i]; }
        qmul = 1.f / sqrtf(sq + 1e-6f) / sqrtf((float)r.d);
        kmul = 1.f / sqrtf(sk + 1e-6f);
        beta = mix_sigmoid(__ldcg(a.beta + (size_t)b * a.ldz + h));
        const int share = (r.d + ranks - 1) / ranks, c0 = rank * share, nc = max(0, min(share, r.d - c0));
        const __nv_bfloat16 *w1 = static_cast<const __nv_bfloat16 *>(a.a2) + (size_t)(h * r.d + c0) * a.ld_a2, *w2 = static_cast<const __nv_bfloat16 *>(a.g2) + (size_t)(h * r.dv + col0) * a.ld_g2;
        float x[4];
        for (int c = warp; c < nc; c += 4 * RS_WARPS) {
            rs_dot4(x, w1, c, RS_WARPS, nc, rs_low, a.ld_a2, lane);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int ch = c0 + c + e * RS_WARPS;
                if (c + e * RS_WARPS < nc && lane < ranks) rs_store_remote(&g[ch], lane, mix_decay(a.a_log[h], x[e] + a.dt_bias[h * r.d + ch]));
            }
        }
        rs_dot4(x, w2, warp, RS_WARPS, ncol, gl, a.ld_g2, lane);
        if (lane < 4 && warp + lane * RS_WARPS < ncol) gate[warp + lane * RS_WARPS] = mix_sigmoid(lane == 0 ? x[0] : (lane == 1 ? x[1] : (lane == 2 ? x[2] : x[3])));
        rs_cluster_sync();
    } else if (WKV || LIGHTNING) {
        for (int i = threadIdx.x; i < r.d; i += RS_THREADS) {
            q[i] = __ldcg(qz + i);
            k[i] = __ldcg(kz + i);
        }
        if (threadIdx.x < ncol) {
            v[threadIdx.x] = __ldcg(vz + threadIdx.x);
            const float z = __ldcg(a.gate + (size_t)b * a.ldz + h * r.dv + col0 + threadIdx.x);
            gate[threadIdx.x] = WKV ? mix_silu(z) : mix_sigmoid(z);
        }
        if (WKV) {
            for (int i = threadIdx.x; i < a.ld_a2; i += RS_THREADS) rs_low[i] = __ldcg(a.a_low + (size_t)b * a.ld_low + i);
            // this CTA's share of the row that the next token mixes with
            const int ctas = ranks * r.H, cta = h * ranks + rank, part = (a.row_n + ctas - 1) / ctas;
            for (int i = cta * part + threadIdx.x; i < min((cta + 1) * part, a.row_n); i += RS_THREADS) a.before[(size_t)b * a.ld_row + i] = __ldcg(a.row + (size_t)b * a.ld_row + i);
        }
        __syncthreads();
        if (WKV) {
            const int share = (r.d + ranks - 1) / ranks, c0 = rank * share, nc = max(0, min(share, r.d - c0));
            const __nv_bfloat16 *w2 = static_cast<const __nv_bfloat16 *>(a.a2) + (size_t)(h * r.d + c0) * a.ld_a2;
            float x[4];
            for (int c = warp; c < nc; c += 4 * RS_WARPS) {
                rs_dot4(x, w2, c, RS_WARPS, nc, rs_low, a.ld_a2, lane);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int ch = c0 + c + e * RS_WARPS;
                    if (c + e * RS_WARPS < nc && lane < ranks) rs_store_remote(&g[ch], lane, expf(-expf(x[e] + a.dt_bias[h * r.d + ch])));
                }
            }
            rs_cluster_sync();
        }
    } else {
        const int half = a.rot_dims / 2;
        kmul = 1.f / sqrtf((float)r.d);
        for (int i = threadIdx.x; i < r.d - half; i += RS_THREADS) {
            if (i < half) {
                float sn, cs;
                sincosf((float)p * a.freq[i], &sn, &cs);
                const float u = __ldcg(qz + i), w = __ldcg(qz + half + i), x = __ldcg(kz + i), y = __ldcg(kz + half + i);
                q[i] = u * cs - w * sn;
                q[half + i] = w * cs + u * sn;
                k[i] = x * cs - y * sn;
                k[half + i] = y * cs + x * sn;
            } else {
                q[half + i] = __ldcg(qz + half + i);
                k[half + i] = __ldcg(kz + half + i);
            }
        }
        if (threadIdx.x < ncol) {
            v[threadIdx.x] = __ldcg(vz + threadIdx.x);
            gate[threadIdx.x] = mix_silu(__ldcg(a.gate + (size_t)b * a.ldz + h * r.dv + col0 + threadIdx.x));
        }
        __syncthreads();
    }
    const RecVec<RPL> kv = rec_read<RPL>(k + lane * RPL), qv = rec_read<RPL>(q + lane * RPL);
    float u[4], po[4];
    if (DELTA) {
        const RecVec<RPL> gv = rec_read<RPL>(g + lane * RPL);
        float pk[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            pk[c] = 0.f;
#pragma unroll
            for (int i = 0; i < RPL; ++i) {
                S[c][i] *= gv.v[i];
                pk[c] = fmaf(S[c][i], kv.v[i] * kmul, pk[c]);
            }
        }
        rec_fold<4>(pk, lane, 16);
        rec_fold<2>(pk, lane, 8);
        const float mine = beta * (v[wcol + (lane >> 3)] - group_sum<8>(pk[0]));
#pragma unroll
        for (int c = 0; c < 4; ++c) u[c] = __shfl_sync(~0u, mine, c * 8);
    } else {
#pragma unroll
        for (int c = 0; c < 4; ++c) u[c] = v[wcol + c];
    }
    const float fixed = LOW ? 1.f : r.decay[h];
    RecVec<RPL> gv = {}, bonus = {};
    if (WKV) {
        gv = rec_read<RPL>(g + lane * RPL);
#pragma unroll
        for (int i = 0; i < RPL; ++i) bonus.v[i] = lane * RPL + i < r.d ? r.bonus[h * r.d + lane * RPL + i] : 0.f;
    }
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        po[c] = 0.f;
#pragma unroll
        for (int i = 0; i < RPL; ++i) {
            if (WKV) {
                const float kv1 = kv.v[i] * u[c];
                po[c] = fmaf(fmaf(bonus.v[i], kv1, S[c][i]), qv.v[i], po[c]);
                S[c][i] = fmaf(gv.v[i], S[c][i], kv1);
                continue;
            }
            S[c][i] = fmaf(kv.v[i] * kmul, u[c], DELTA ? S[c][i] : fixed * S[c][i]);
            po[c] = fmaf(S[c][i], qv.v[i] * qmul, po[c]);
        }
    }
#pragma unroll
    for (int c = 0; c < 4; ++c)
        if (wcol + c < ncol)
#pragma unroll
            for (int i = 0; i < RPL; ++i) st[(size_t)c * DP + i] = S[c][i];
    rec_fold<4>(po, lane, 16);
    rec_fold<2>(po, lane, 8);
    po[0] = group_sum<8>(po[0]);
    if ((lane & 7) == 0) o[wcol + (lane >> 3)] = po[0];      // columns past ncol: zero state, zero
    __syncthreads();
    if (warp == 0) {
        const float ss = group_sum<32>(o[lane] * o[lane]);
        if (lane < ranks) rs_store_remote(&part[rank], lane, ss);
    }
    rs_cluster_sync();
    float ss = 0.f;
    for (int i = 0; i < ranks; ++i) ss += part[i];
    if (threadIdx.x < ncol) {
        const float rs = LIGHTNING ? a.mul : 1.f / sqrtf(ss / (float)r.dv + a.eps);
        const float w = !a.head_norm ? 1.f : a.head_norm[(WKV || LIGHTNING ? h * r.dv : 0) + col0 + threadIdx.x];
        mix_store(a.dst, (size_t)b * a.ldd + h * r.dv + col0 + threadIdx.x, o[threadIdx.x] * rs * w * gate[threadIdx.x], a.act_f32);
    }
    if (LIGHTNING) {
        if (rank == 0 && threadIdx.x == 0) a.part[(size_t)b * r.H + h] = ss;
        if (a.ready) pdl_wait();                              // the launch after this one relies on the one before it, too
    }
}

template <int RPL, int KIND>
static int rs_launch(const RecurStep *a, int B, const int *pos, cudaStream_t st)
{
    const int ranks = (a->r.dv + RS_COLS - 1) / RS_COLS;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(ranks, a->r.H, B);
    cfg.blockDim = dim3(RS_THREADS);
    cfg.dynamicSmemBytes = KIND == STEP_DELTA || KIND == STEP_WKV ? (size_t)(a->ld_a2 + a->ld_g2) * sizeof(float) : 0;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = ranks;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = ckb_tune_get("pdl", 1) ? 2 : 1;
    if (ckb_check_cuda((int)cudaLaunchKernelEx(&cfg, recur_step_kernel<RPL, KIND>, *a, B, pos), "recur_step")) return CKB_ERR_CUDA;
    return ckb_check_launch("recur_step");
}

template <int RPL>
static int rs_pick(const RecurStep *a, int B, const int *pos, cudaStream_t st)
{
    switch (a->kind) {
        case STEP_DELTA: return rs_launch<RPL, STEP_DELTA>(a, B, pos, st);
        case STEP_WKV: return rs_launch<RPL, STEP_WKV>(a, B, pos, st);
        case STEP_LIGHTNING: return rs_launch<RPL, STEP_LIGHTNING>(a, B, pos, st);
        default: return rs_launch<RPL, STEP_RETENTION>(a, B, pos, st);
    }
}

}  // namespace ckb

using namespace ckb;

extern "C" int ckb_recur_step_takes(int d, int dv, int ld_a2, int ld_g2) { return ckb_recur_dp(d) != 0 && dv <= 8 * RS_COLS && ld_a2 + ld_g2 <= 8192; }

extern "C" int ckb_launch_recur_step(const RecurStep *a, int B, const int *pos, void *stream)
{
    cudaStream_t st = ckb_stream(stream);
    if (!ckb_recur_step_takes(a->r.d, a->r.dv, a->ld_a2, a->ld_g2)) return ckb_fail(CKB_ERR_LIMIT, "recur_step: heads of %d x %d, low ranks of %d + %d", a->r.d, a->r.dv, a->ld_a2, a->ld_g2);
    switch (ckb_recur_dp(a->r.d)) {
        case 32: return rs_pick<1>(a, B, pos, st);
        case 64: return rs_pick<2>(a, B, pos, st);
        case 128: return rs_pick<4>(a, B, pos, st);
        default: return rs_pick<8>(a, B, pos, st);
    }
}
