// Linear recurrences over time, one fp32 state matrix per head: fixed decay (S = a S + k v^T) or gated delta rule
// (S = g S; u = beta (v - S^T k); S = S + k u^T), read out as S^T q after the token's own write.
//
// The columns of S (one per value channel) do not interact, so a CTA takes 16 columns of one head of one sequence and walks the tokens
// in order; eight lanes share a column, each with NR of its rows in registers (rows 32 i + 4 lane + 0..3, so that a lane reads a token's
// key, query and decay 16 bytes at a time).  Per token and column: S *= g, two dot products with the decayed state (with k and with q),
// one three-step butterfly over the eight lanes, S += k u; the read-out is S_decayed^T q + (k.q) u, so that both dot products are
// reduced together.  Tokens are staged in shared memory REC_TOKENS at a time by cp.async, one batch ahead.  The decode step is the same
// kernel with one token: it then streams the state once, 16 bytes a lane.
#include "device_common.cuh"
#include "launch.h"
#include "mixers.h"
#include "pdl.cuh"
#include "runtime.h"

namespace ckb {

constexpr int REC_COLS = 16, REC_TOKENS = 16, REC_THREADS = REC_COLS * 8;

__device__ __forceinline__ void cp_async4(uint32_t dst, const void *src) { asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }

// `n` floats of REC_TOKENS (or fewer) rows, one row every `row_stride` floats, into rows of `width` floats
__device__ __forceinline__ void rec_stage(float *dst, int width, const float *src, size_t row_stride, int n, int tokens)
{
    if ((n & 3) == 0 && ((reinterpret_cast<uintptr_t>(src) | row_stride * 4) & 15) == 0) {
        const int q = n >> 2;
        for (int i = threadIdx.x; i < tokens * q; i += REC_THREADS) cp_async16(smem_u32(dst + (i / q) * width + (i % q) * 4), src + (i / q) * row_stride + (i % q) * 4);
    } else {
        for (int i = threadIdx.x; i < tokens * n; i += REC_THREADS) cp_async4(smem_u32(dst + (i / n) * width + i % n), src + (i / n) * row_stride + i % n);
    }
}

template <int NR, bool DELTA>
__global__ __launch_bounds__(REC_THREADS) void recur_rows_kernel(const __grid_constant__ RecurRows a, int T, int B)
{
    constexpr int DP = NR * 8, NG = NR / 4, VECS = DELTA ? 3 : 2, BUF = REC_TOKENS * (VECS * DP + REC_COLS + 1);
    extern __shared__ __align__(16) float rec_sm[];          // two of { k, q, (g), v, beta } and the k.q of the batch in work
    float *kq = rec_sm + 2 * BUF;
    const int col0 = blockIdx.x * REC_COLS, h = blockIdx.y, b = blockIdx.z, kh = h / (a.H / a.G);
    const int lane = threadIdx.x & 7, cl = threadIdx.x >> 3, col = col0 + cl, ncol = min(REC_COLS, a.dv - col0);
    const bool live = cl < ncol;
    float *st = a.state + (((size_t)b * a.H + h) * a.dv + col) * DP + lane * 4;
    pdl_wait();
    pdl_trigger();
    float S[NR];
#pragma unroll
    for (int i = 0; i < NG; ++i) {
        const float4 v = live ? __ldcg(reinterpret_cast<const float4 *>(st + i * 32)) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[4 * i] = v.x; S[4 * i + 1] = v.y; S[4 * i + 2] = v.z; S[4 * i + 3] = v.w;
    }
    // rows past d and columns past dv stay zero in both buffers
    for (int i = threadIdx.x; i < 2 * BUF; i += REC_THREADS) rec_sm[i] = 0.f;
    __syncthreads();
    const float fixed = DELTA ? 0.f : a.decay[h];
    auto stage = [&](int buf, int t0) {
        const int n = min(REC_TOKENS, T - t0);
        const size_t row = (size_t)t0 * B + b;
        float *base = rec_sm + buf * BUF;
        rec_stage(base, DP, a.k + row * a.ldk + kh * a.d, (size_t)B * a.ldk, a.d, n);
        rec_stage(base + REC_TOKENS * DP, DP, a.q + row * a.ldq + kh * a.d, (size_t)B * a.ldq, a.d, n);
        if (DELTA) rec_stage(base + 2 * REC_TOKENS * DP, DP, a.g + row * a.ldg + h * a.d, (size_t)B * a.ldg, a.d, n);
        rec_stage(base + VECS * REC_TOKENS * DP, REC_COLS, a.v + row * a.ldv + h * a.dv + col0, (size_t)B * a.ldv, ncol, n);
        if (DELTA) rec_stage(base + REC_TOKENS * (VECS * DP + REC_COLS), 1, a.beta + row * a.ldb + h, (size_t)B * a.ldb, 1, n);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    int buf = 0;
    for (int t0 = 0; t0 < T; t0 += REC_TOKENS, buf ^= 1) {
        const int n = min(REC_TOKENS, T - t0);
        if (t0 + REC_TOKENS < T) {
            stage(buf ^ 1, t0 + REC_TOKENS);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float *ks = rec_sm + buf * BUF, *qs = ks + REC_TOKENS * DP, *gs = qs + REC_TOKENS * DP, *vs = ks + VECS * REC_TOKENS * DP, *bs = vs + REC_TOKENS * REC_COLS;
        if (DELTA) {                                          // k.q of token cl, by the eight lanes of column cl
            float p = 0.f;
#pragma unroll
            for (int i = 0; i < NG; ++i) {
                const float4 k = *reinterpret_cast<const float4 *>(ks + cl * DP + i * 32 + lane * 4), q = *reinterpret_cast<const float4 *>(qs + cl * DP + i * 32 + lane * 4);
                p = fmaf(k.x, q.x, fmaf(k.y, q.y, fmaf(k.z, q.z, fmaf(k.w, q.w, p))));
            }
            p = group_sum<8>(p);
            if (lane == 0) kq[cl] = p;
            __syncthreads();
        }
        float *out = a.o + ((size_t)t0 * B + b) * a.ldo + h * a.dv + col;
        for (int t = 0; t < n; ++t) {
            float4 k[NG], q[NG];
#pragma unroll
            for (int i = 0; i < NG; ++i) {
                k[i] = *reinterpret_cast<const float4 *>(ks + t * DP + i * 32 + lane * 4);
                q[i] = *reinterpret_cast<const float4 *>(qs + t * DP + i * 32 + lane * 4);
            }
            const float v = vs[t * REC_COLS + cl];
            float o;
            if (DELTA) {
                float pk[2] = {0.f, 0.f}, pq[2] = {0.f, 0.f};
#pragma unroll
                for (int i = 0; i < NG; ++i) {
                    const float4 g = *reinterpret_cast<const float4 *>(gs + t * DP + i * 32 + lane * 4);
                    S[4 * i] *= g.x; S[4 * i + 1] *= g.y; S[4 * i + 2] *= g.z; S[4 * i + 3] *= g.w;
                    pk[i & 1] = fmaf(S[4 * i], k[i].x, pk[i & 1]); pq[i & 1] = fmaf(S[4 * i], q[i].x, pq[i & 1]);
                    pk[i & 1] = fmaf(S[4 * i + 1], k[i].y, pk[i & 1]); pq[i & 1] = fmaf(S[4 * i + 1], q[i].y, pq[i & 1]);
                    pk[i & 1] = fmaf(S[4 * i + 2], k[i].z, pk[i & 1]); pq[i & 1] = fmaf(S[4 * i + 2], q[i].z, pq[i & 1]);
                    pk[i & 1] = fmaf(S[4 * i + 3], k[i].w, pk[i & 1]); pq[i & 1] = fmaf(S[4 * i + 3], q[i].w, pq[i & 1]);
                }
                const float sk = group_sum<8>(pk[0] + pk[1]), sq = group_sum<8>(pq[0] + pq[1]);
                const float u = bs[t] * (v - sk);
                o = fmaf(kq[t], u, sq);
#pragma unroll
                for (int i = 0; i < NG; ++i) {
                    S[4 * i] = fmaf(k[i].x, u, S[4 * i]); S[4 * i + 1] = fmaf(k[i].y, u, S[4 * i + 1]);
                    S[4 * i + 2] = fmaf(k[i].z, u, S[4 * i + 2]); S[4 * i + 3] = fmaf(k[i].w, u, S[4 * i + 3]);
                }
            } else {
                float pq[2] = {0.f, 0.f};
#pragma unroll
                for (int i = 0; i < NG; ++i) {
                    S[4 * i] = fmaf(k[i].x, v, fixed * S[4 * i]); pq[i & 1] = fmaf(S[4 * i], q[i].x, pq[i & 1]);
                    S[4 * i + 1] = fmaf(k[i].y, v, fixed * S[4 * i + 1]); pq[i & 1] = fmaf(S[4 * i + 1], q[i].y, pq[i & 1]);
                    S[4 * i + 2] = fmaf(k[i].z, v, fixed * S[4 * i + 2]); pq[i & 1] = fmaf(S[4 * i + 2], q[i].z, pq[i & 1]);
                    S[4 * i + 3] = fmaf(k[i].w, v, fixed * S[4 * i + 3]); pq[i & 1] = fmaf(S[4 * i + 3], q[i].w, pq[i & 1]);
                }
                o = group_sum<8>(pq[0] + pq[1]);
            }
            if (lane == 0 && live) out[(size_t)t * B * a.ldo] = o;
        }
        __syncthreads();                                      // before the next batch overwrites this buffer
    }
    if (live)
#pragma unroll
        for (int i = 0; i < NG; ++i) *reinterpret_cast<float4 *>(st + i * 32) = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
}

template <int NR, bool DELTA>
static int rec_launch(const RecurRows *a, int T, int B, cudaStream_t st)
{
    constexpr int VECS = DELTA ? 3 : 2;
    const int smem = (2 * REC_TOKENS * (VECS * NR * 8 + REC_COLS + 1) + REC_TOKENS) * (int)sizeof(float);
    static bool attr = false;
    if (!attr) {
        if (ckb_check_cuda((int)cudaFuncSetAttribute(recur_rows_kernel<NR, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), "recur_rows smem")) return CKB_ERR_CUDA;
        attr = true;
    }
    return launch_pdl("recur_rows", recur_rows_kernel<NR, DELTA>, dim3((a->dv + REC_COLS - 1) / REC_COLS, a->H, B), dim3(REC_THREADS), (size_t)smem, st, *a, T, B);
}

}  // namespace ckb

using namespace ckb;

extern "C" int ckb_recur_dp(int d) { return d <= 0 || d > 256 ? 0 : (d <= 32 ? 32 : (d <= 64 ? 64 : (d <= 128 ? 128 : 256))); }

extern "C" int ckb_launch_recur_rows(const RecurRows *a, int T, int B, void *stream)
{
    cudaStream_t st = ckb_stream(stream);
    const bool delta = a->g != nullptr;
    switch (ckb_recur_dp(a->d)) {
        case 32: return delta ? rec_launch<4, true>(a, T, B, st) : rec_launch<4, false>(a, T, B, st);
        case 64: return delta ? rec_launch<8, true>(a, T, B, st) : rec_launch<8, false>(a, T, B, st);
        case 128: return delta ? rec_launch<16, true>(a, T, B, st) : rec_launch<16, false>(a, T, B, st);
        case 256: return delta ? rec_launch<32, true>(a, T, B, st) : rec_launch<32, false>(a, T, B, st);
    }
    return ckb_fail(CKB_ERR_SHAPE, "recurrence: head size %d (at most 256)", a->d);
}
