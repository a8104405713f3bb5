// Linear recurrences over time, one fp32 state matrix per head: fixed decay (S = a S + k v^T) or gated delta rule
// (S = g S; u = beta (v - S^T k); S = S + k u^T), read out as S^T q after the token's own write; or a decay per row with a bonus for the
// current token, read out before the write (o = (S + diag(bonus) k v^T)^T q; S = g S + k v^T).
//
// The columns of S (one per value channel) do not interact, so a warp takes two or four columns of one head of one sequence and walks
// the tokens in order, the rows spread over its lanes (RPL consecutive rows each, in registers).  Every lane then reads its own part of
// a token's key, query and decay from shared memory, one token ahead and once for its columns; the arithmetic is packed fp32 (two rows
// an instruction).  Per token the delta rule needs one sum over the lanes per column before it can update (S^T k): a butterfly for all
// columns at once, then u goes back to all lanes.  The read-outs wait in registers until 32 of them are there and are then summed over
// the lanes together, one shuffle per value.  Tokens are staged REC_TOKENS at a time by cp.async, one batch ahead, for the 16 columns of
// a CTA.  Short passes sum their read-outs token by token.
#include "device_common.cuh"
#include "launch.h"
#include "mixer_lanes.cuh"
#include "mixers.h"
#include "pdl.cuh"
#include "runtime.h"

namespace ckb {

enum { REC_FIXED = 0, REC_DELTA, REC_BONUS };
constexpr int REC_COLS = 16, REC_TOKENS = 16, REC_BLOCK = 8;

__device__ __forceinline__ void cp_async4(uint32_t dst, const void *src) { asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }

// `n` floats of REC_TOKENS (or fewer) rows, one row every `row_stride` floats, into rows of `width` floats
template <int REC_THREADS>
__device__ __forceinline__ void rec_stage(float *dst, int width, const float *src, size_t row_stride, int n, int tokens)
{
    if ((n & 3) == 0 && ((reinterpret_cast<uintptr_t>(src) | row_stride * 4) & 15) == 0) {
        const int q = n >> 2;
        if ((q & (q - 1)) == 0) {                             // no divisions where the row length is a power of two
            const int sh = 31 - __clz(q);
            for (int i = threadIdx.x; i < tokens << sh; i += REC_THREADS)
                cp_async16(smem_u32(dst + (i >> sh) * width + (i & (q - 1)) * 4), src + (i >> sh) * row_stride + (i & (q - 1)) * 4);
        } else {
            for (int i = threadIdx.x; i < tokens * q; i += REC_THREADS) cp_async16(smem_u32(dst + (i / q) * width + (i % q) * 4), src + (i / q) * row_stride + (i % q) * 4);
        }
    } else {
        for (int i = threadIdx.x; i < tokens * n; i += REC_THREADS) cp_async4(smem_u32(dst + (i / n) * width + i % n), src + (i / n) * row_stride + i % n);
    }
}

// WC: columns per warp.  TB: tokens whose read-outs are summed together (32 / WC of them fill a warp), or 1 for short passes
template <int RPL, int MODE, int WC, int TB>
__global__ __launch_bounds__(REC_COLS / WC * 32) void recur_rows_kernel(const __grid_constant__ RecurRows a, int T, int B)
{
    constexpr bool DELTA = MODE == REC_DELTA, GATED = MODE != REC_FIXED;
    constexpr int REC_THREADS = REC_COLS / WC * 32, SHIFT = WC == 4 ? 3 : 4;      // lanes >> SHIFT = column, in the sum over the lanes
    constexpr int DP = RPL * 32, VECS = GATED ? 3 : 2, BUF = REC_TOKENS * (VECS * DP + REC_COLS + 1);
    constexpr int OFF_Q = REC_TOKENS * DP, OFF_G = 2 * REC_TOKENS * DP, OFF_V = VECS * REC_TOKENS * DP, OFF_B = OFF_V + REC_TOKENS * REC_COLS;
    extern __shared__ __align__(16) float rec_sm[];          // two of { k, q, (g), v, beta }
    const int col0 = blockIdx.x * REC_COLS, h = blockIdx.y, b = blockIdx.z, kh = h / (a.H / a.G), ncol = min(REC_COLS, a.dv - col0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wcol = warp * WC;
    float *st = a.state + (((size_t)b * a.H + h) * a.dv + col0 + wcol) * DP + lane * RPL;
    pdl_wait();
    if (TB == 1) pdl_trigger();                               // a long pass keeps the SMs to itself
    constexpr int NP = RecPairs<RPL>::N;
    float2 S[WC][NP];
#pragma unroll
    for (int c = 0; c < WC; ++c) {
        RecVec<RPL> r = {};
        if (wcol + c < ncol) r = rec_read<RPL>(st + (size_t)c * DP);
        const RecPairs<RPL> x = rec_pairs(r);
#pragma unroll
        for (int i = 0; i < NP; ++i) S[c][i] = x.v[i];
    }
    RecPairs<RPL> bonus = {};
    if (MODE == REC_BONUS) {
        RecVec<RPL> r;
#pragma unroll
        for (int i = 0; i < RPL; ++i) r.v[i] = lane * RPL + i < a.d ? a.bonus[h * a.d + lane * RPL + i] : 0.f;
        bonus = rec_pairs(r);
    }
    // what no token fills stays neutral: zero rows past d and columns past dv; of a last, short batch of tokens zero keys, queries and
    // beta, and decays of one
    for (int i = threadIdx.x; i < 2 * BUF; i += REC_THREADS) rec_sm[i] = GATED && i % BUF >= OFF_G && i % BUF < OFF_V ? 1.f : 0.f;
    __syncthreads();
    const float fixed = GATED ? 0.f : a.decay[h];
    auto stage = [&](int buf, int t0) {
        const int n = min(REC_TOKENS, T - t0);
        const size_t row = (size_t)t0 * B + b;
        float *base = rec_sm + buf * BUF;
        rec_stage<REC_THREADS>(base, DP, a.k + row * a.ldk + kh * a.d, (size_t)B * a.ldk, a.d, n);
        rec_stage<REC_THREADS>(base + OFF_Q, DP, a.q + row * a.ldq + kh * a.d, (size_t)B * a.ldq, a.d, n);
        if (GATED) rec_stage<REC_THREADS>(base + OFF_G, DP, a.g + row * a.ldg + h * a.d, (size_t)B * a.ldg, a.d, n);
        rec_stage<REC_THREADS>(base + OFF_V, REC_COLS, a.v + row * a.ldv + h * a.dv + col0, (size_t)B * a.ldv, ncol, n);
        if (DELTA) rec_stage<REC_THREADS>(base + OFF_B, 1, a.beta + row * a.ldb + h, (size_t)B * a.ldb, 1, n);
        if (n < REC_TOKENS && T > REC_TOKENS) {               // tokens past the end of a buffer that held others
            for (int i = n * DP + threadIdx.x; i < REC_TOKENS * DP; i += REC_THREADS) {
                base[i] = 0.f;
                base[OFF_Q + i] = 0.f;
                if (GATED) base[OFF_G + i] = 1.f;
            }
            for (int i = n * REC_COLS + threadIdx.x; i < REC_TOKENS * REC_COLS; i += REC_THREADS) base[OFF_V + i] = 0.f;
            if (DELTA) for (int i = n + threadIdx.x; i < REC_TOKENS; i += REC_THREADS) base[OFF_B + i] = 0.f;
        }
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
        const float *base = rec_sm + buf * BUF, *ks = base + lane * RPL, *vs = base + OFF_V + wcol, *bs = base + OFF_B;
        RecPairs<RPL> kn, qn, gn;
        auto fetch = [&](int t) {
            kn = rec_pairs(rec_read<RPL>(ks + t * DP));
            qn = rec_pairs(rec_read<RPL>(ks + OFF_Q + t * DP));
            if (GATED) gn = rec_pairs(rec_read<RPL>(ks + OFF_G + t * DP));
        };
        fetch(0);
        for (int tb = 0; tb < n; tb += TB) {
            float po[TB * WC];                                // read-outs, this lane's rows: [token][column]
#pragma unroll
            for (int j = 0; j < TB; ++j) {
                const int t = tb + j;
                const RecPairs<RPL> k = kn, q = qn, g = gn;
                if (t + 1 < REC_TOKENS) fetch(t + 1);         // the next token's rows are on their way during this one's sums
                float u[WC];
                if (DELTA) {
                    float pk[WC];
#pragma unroll
                    for (int c = 0; c < WC; ++c) {
                        float2 p = make_float2(0.f, 0.f);
#pragma unroll
                        for (int i = 0; i < NP; ++i) {
                            S[c][i] = mul2(S[c][i], g.v[i]);
                            p = fma2(S[c][i], k.v[i], p);
                        }
                        pk[c] = p.x + p.y;
                    }
                    if (WC == 4) rec_fold<WC>(pk, lane, 16);
                    rec_fold<2>(pk, lane, WC == 4 ? 8 : 16);
                    const float sum = group_sum<(1 << SHIFT)>(pk[0]);       // of column lane >> SHIFT
                    const float mine = bs[t] * (vs[t * REC_COLS + (lane >> SHIFT)] - sum);
#pragma unroll
                    for (int c = 0; c < WC; ++c) u[c] = __shfl_sync(~0u, mine, c << SHIFT);
                } else {
#pragma unroll
                    for (int c = 0; c < WC; ++c) u[c] = vs[t * REC_COLS + c];
                }
                const float keep = TB == 1 || t < n ? fixed : 1.f;            // tokens past the end leave the state alone
#pragma unroll
                for (int c = 0; c < WC; ++c) {
                    float2 o = make_float2(0.f, 0.f);
                    const float2 u2 = make_float2(u[c], u[c]);
#pragma unroll
                    for (int i = 0; i < NP; ++i) {
                        if (MODE == REC_BONUS) {
                            const float2 kv = mul2(k.v[i], u2);
                            o = fma2(fma2(bonus.v[i], kv, S[c][i]), q.v[i], o);
                            S[c][i] = fma2(g.v[i], S[c][i], kv);
                        } else {
                            S[c][i] = fma2(k.v[i], u2, DELTA ? S[c][i] : mul2(make_float2(keep, keep), S[c][i]));
                            o = fma2(S[c][i], q.v[i], o);
                        }
                    }
                    po[j * WC + c] = o.x + o.y;
                }
            }
            if (TB > 1) {                                     // 32 values: lane = token * WC + column
                constexpr int N = TB > 1 ? 32 : 2;
                static_assert(TB == 1 || TB * WC == 32, "one value per lane");
                rec_fold<N>(po, lane, 16);
                rec_fold<N / 2>(po, lane, 8);
                rec_fold<N / 4>(po, lane, 4);
                rec_fold<N / 8>(po, lane, 2);
                rec_fold<N / 16>(po, lane, 1);
                const int t = tb + lane / WC, c = wcol + lane % WC;
                if (t < n && c < ncol) a.o[((size_t)(t0 + t) * B + b) * a.ldo + h * a.dv + col0 + c] = po[0];
            } else {
                if (WC == 4) rec_fold<WC>(po, lane, 16);
                rec_fold<2>(po, lane, WC == 4 ? 8 : 16);
                const float o = group_sum<(1 << SHIFT)>(po[0]);
                const int c = wcol + (lane >> SHIFT);
                if ((lane & ((1 << SHIFT) - 1)) == 0 && c < ncol) a.o[((size_t)(t0 + tb) * B + b) * a.ldo + h * a.dv + col0 + c] = o;
            }
        }
        __syncthreads();                                      // before the next batch overwrites this buffer
    }
#pragma unroll
    for (int c = 0; c < WC; ++c)
        if (wcol + c < ncol)
#pragma unroll
            for (int i = 0; i < RPL; ++i) st[(size_t)c * DP + i] = i & 1 ? S[c][i / 2].y : S[c][i / 2].x;
}

template <int RPL, int MODE, int WC, int TB>
static int rec_launch_tb(const RecurRows *a, int T, int B, cudaStream_t st)
{
    constexpr int VECS = MODE != REC_FIXED ? 3 : 2, THREADS = REC_COLS / WC * 32;
    const int smem = 2 * REC_TOKENS * (VECS * RPL * 32 + REC_COLS + 1) * (int)sizeof(float);
    static bool attr = false;
    if (!attr) {
        if (ckb_check_cuda((int)cudaFuncSetAttribute(recur_rows_kernel<RPL, MODE, WC, TB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), "recur_rows smem")) return CKB_ERR_CUDA;
        attr = true;
    }
    const dim3 grid((a->dv + REC_COLS - 1) / REC_COLS, a->H, B);
    if (TB == 1) return launch_pdl("recur_rows", recur_rows_kernel<RPL, MODE, WC, TB>, grid, dim3(THREADS), (size_t)smem, st, *a, T, B);
    return launch_plain("recur_rows", recur_rows_kernel<RPL, MODE, WC, TB>, grid, dim3(THREADS), (size_t)smem, st, *a, T, B);
}
template <int RPL, int MODE>
static int rec_launch(const RecurRows *a, int T, int B, cudaStream_t st)
{
    if (T < REC_BLOCK) return rec_launch_tb<RPL, MODE, 2, 1>(a, T, B, st);
    // two columns per warp measured as fast as four until the SMs are full of warps; then the fewer shared-memory reads of four win
    return (long long)a->H * a->dv * B >= 8192 ? rec_launch_tb<RPL, MODE, 4, 8>(a, T, B, st) : rec_launch_tb<RPL, MODE, 2, 16>(a, T, B, st);
}

template <int RPL>
static int rec_pick(const RecurRows *a, int T, int B, cudaStream_t st)
{
    if (!a->g) return rec_launch<RPL, REC_FIXED>(a, T, B, st);
    return a->bonus ? rec_launch<RPL, REC_BONUS>(a, T, B, st) : rec_launch<RPL, REC_DELTA>(a, T, B, st);
}

}  // namespace ckb

using namespace ckb;

extern "C" int ckb_recur_dp(int d) { return d <= 0 || d > 256 ? 0 : (d <= 32 ? 32 : (d <= 64 ? 64 : (d <= 128 ? 128 : 256))); }

extern "C" int ckb_launch_recur_rows(const RecurRows *a, int T, int B, void *stream)
{
    cudaStream_t st = ckb_stream(stream);
    switch (ckb_recur_dp(a->d)) {
        case 32: return rec_pick<1>(a, T, B, st);
        case 64: return rec_pick<2>(a, T, B, st);
        case 128: return rec_pick<4>(a, T, B, st);
        case 256: return rec_pick<8>(a, T, B, st);
    }
    return ckb_fail(CKB_ERR_SHAPE, "recurrence: head size %d (at most 256)", a->d);
}
