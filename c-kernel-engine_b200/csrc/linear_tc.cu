// y = x W^T for bfloat16 weights and activations on the 5th-generation tensor cores, fp32 accumulation in tensor memory.
//
// The weight rows are the M = 128 operand (one TMEM lane each) and the tokens the N operand (a column each), so a finished accumulator
// column is 32 consecutive outputs of one token per warp: stores are coalesced, a 32-row block lies in one segment (linear.h), and the
// token tile is as wide as suits the portion, up to 256.  Both operands come as 128-byte-swizzled tiled bulk copies, 64 columns a stage.
//
// Persistent CTAs of 256 threads: warp 0 loads, warp 1 issues (one elected lane each), warps 4-7 drain one accumulator buffer while the
// next tile fills the other.  Tiles go row block by row block with the token tiles innermost: CTAs that run side by side share weight
// tiles in L2.  Every wait is bounded; a timeout sets the device error word and a flag that ends the other roles, copies in flight
// are waited for (again bounded) and the tensor memory is freed.
#include <cuda.h>
#include <string.h>

#include "device_common.cuh"
#include "launch.h"
#include "linear_epilogue.cuh"
#include "pdl.cuh"
#include "runtime.h"
#include "tcgen05.cuh"

namespace ckb {

constexpr int LT_ROWS = 128, LT_K = 64, LT_A_BYTES = LT_ROWS * LT_K * 2, LT_THREADS = 256;

constexpr int LT_MAX_WIDTH = 256, LT_MAX_STAGES = 8, LT_BARS = (2 * LT_MAX_STAGES + 5) * 8 + 16;
constexpr int LT_SMEM = 199 * 1024;           // of stages; the rest is for the small kernels that start beside it
// bf16 x bf16 -> f32, both operands K-major, M = 128; N is added
constexpr uint32_t LT_IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(LT_ROWS >> 4) << 24);

// tokens of a tile, and what follows from that
struct LtTile {
    int width, stage, stages, columns;       // bytes and number of stages; tensor memory columns of one accumulator
    constexpr explicit LtTile(int w) : width(w), stage(LT_A_BYTES + w * LT_K * 2), stages(LT_SMEM / stage < LT_MAX_STAGES ? LT_SMEM / stage : LT_MAX_STAGES), columns(16)
    {
        while (columns < w) columns *= 2;
    }
    int smem() const { return stages * stage + LT_BARS + 1024; }      // + alignment of the first stage
};

// shared-memory descriptor of a K-major tile in 128-byte swizzle: 8-row groups 1024 bytes apart
__device__ __forceinline__ uint64_t lt_desc(uint32_t addr)
{
    return (uint64_t)((addr & 0x3FFFFu) >> 4) | (1ull << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}

__device__ __forceinline__ void lt_tma(uint32_t dst, const CUtensorMap *map, int x, int y, uint32_t bar)
{
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                 ::"r"(dst), "l"(map), "r"(x), "r"(y), "r"(bar) : "memory");
}

// NT: width of the tile where it is known at compile time, 0: from `tile_arg`.  MORE: there are lead rows, or some segment makes something
// of its sums or reads an input of its own
template <int NT, bool MORE>
__global__ __launch_bounds__(LT_THREADS, 1) void linear_tc_kernel(const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap xmap, int rows, int ksteps,
                                                                  int tokens, int lead, const LtTile tile_arg, const __grid_constant__ LinSegs segs, int *err)
{
    const LtTile tl = NT ? LtTile(NT) : tile_arg;
    const int width = tl.width, stages = tl.stages;
    if (!MORE) lead = 0;
    extern __shared__ uint8_t lt_raw[];
    uint8_t *sm = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(lt_raw) + 1023) & ~(uintptr_t)1023);
    const uint32_t base = smem_u32(sm), bars = base + stages * tl.stage;
    const uint32_t full = bars, empty = bars + stages * 8, tfull = empty + stages * 8, tempty = tfull + 16, drain = tempty + 16;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(sm + stages * tl.stage + (2 * stages + 5) * 8);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int ttiles = (tokens + lead + width - 1) / width, tiles = ((rows + LT_ROWS - 1) / LT_ROWS) * ttiles;
    if (threadIdx.x == 0) {
        for (int i = 0; i < stages; ++i) { mbar_init(full + i * 8, 1); mbar_init(empty + i * 8, 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(tfull + i * 8, 1); mbar_init(tempty + i * 8, 4); }
        mbar_init(drain, 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 2) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(2 * tl.columns));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    pdl_wait();
    if (warp == 0) {
        if (tc_elect_one()) {
            int s = 0, issued = 0;
            uint32_t ph = 0, st = base, bar = full;           // of stage s; its `empty` barrier is `stages` further on
            bool ok = true;
            for (int tile = blockIdx.x; ok && tile < tiles; tile += gridDim.x) {
                const int r0 = tile / ttiles * LT_ROWS, t0 = tile % ttiles * width, in = MORE ? lin_find(segs, r0) : -1, x0 = in < 0 ? 0 : segs.s[in].x0;
                for (int k = 0; k < ksteps; ++k) {
                    if (!mbar_try_wait(bar + stages * 8, ph ^ 1) && (*abort_flag || !mbar_wait_spin(bar + stages * 8, ph ^ 1))) { ok = false; break; }
                    mbar_arrive_expect_tx(bar, tl.stage);
                    lt_tma(st, &wmap, k * LT_K, r0, bar);
                    lt_tma(st + LT_A_BYTES, &xmap, x0 + k * LT_K, t0, bar);
                    ++issued;
                    st += tl.stage;
                    bar += 8;
                    if (++s == stages) { s = 0; st = base; bar = full; ph ^= 1; }
                }
            }
            if (!ok) {
                *abort_flag = 1;
                atomicExch(err, DEV_ERR_EMPTY_WAIT);
                for (int i = 0; i < stages && i < issued; ++i) {          // copies in flight land before the block ends
                    if (s == 0) { s = stages; ph ^= 1; }
                    --s;
                    mbar_wait_spin(full + s * 8, ph);
                }
            }
        }
    } else if (warp == 1) {
        if (tc_elect_one()) {
            int s = 0, u = 0;
            uint32_t ph = 0, st = base, bar = full;
            const uint32_t idesc = LT_IDESC | (uint32_t)(width >> 3) << 17;
            bool ok = true;
            for (int tile = blockIdx.x; ok && tile < tiles; tile += gridDim.x, ++u) {
                const uint32_t d = tmem + (u & 1) * tl.columns;
                if (*abort_flag || !mbar_wait_spin(tempty + (u & 1) * 8, ((u >> 1) & 1) ^ 1)) { ok = false; break; }
                tc_fence_after();
                for (int k = 0; k < ksteps; ++k) {
                    if (!mbar_wait_spin(bar, ph)) { ok = false; break; }
                    tc_fence_after();
                    const uint64_t da = lt_desc(st), db = da + (LT_A_BYTES >> 4);
#pragma unroll
                    for (int kk = 0; kk < LT_K / 16; ++kk) tc_mma(d, da + kk * 2, db + kk * 2, idesc, (k | kk) != 0);
                    tc_commit(bar + stages * 8);
                    st += tl.stage;
                    bar += 8;
                    if (++s == stages) { s = 0; st = base; bar = full; ph ^= 1; }
                }
                if (ok) tc_commit(tfull + (u & 1) * 8);
            }
            if (!ok) {
                *abort_flag = 1;
                atomicExch(err, DEV_ERR_FULL_WAIT);
                tc_commit(drain);                              // products in flight finish before the tensor memory is freed
                mbar_wait_spin(drain, 0);
            }
        }
    } else if (warp >= 4) {
        const int q = warp & 3;
        int u = 0;
        for (int tile = blockIdx.x; tile < tiles; tile += gridDim.x, ++u) {
            const int r0 = tile / ttiles * LT_ROWS + q * 32, t0 = tile % ttiles * width;
            const int seg = r0 < rows ? lin_find(segs, r0) : -1;
            const bool there = !*abort_flag && mbar_wait_spin(tfull + (u & 1) * 8, (u >> 1) & 1);
            if (!__all_sync(~0u, there)) {
                if (lane == 0) { *abort_flag = 1; atomicExch(err, DEV_ERR_MMA_WAIT); }
                break;
            }
            tc_fence_after();
            if (seg >= 0) {
                const LinSeg &sg = segs.s[seg];
                const int kind = sg.kind, col = r0 - sg.row0 + lane, act = MORE ? segs.act : ACT_BF16;
                const uint32_t src = tmem + (u & 1) * tl.columns + ((uint32_t)(q * 32) << 16);
                const int nt = min(width, tokens + lead - t0);
#pragma unroll 1
                for (int c = 0; c < nt; c += 16) {
                    uint32_t r[16];
                    tc_ld16(src + c, r);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                    int tok = t0 + c - lead, left = nt - c;           // the 16 columns: tokens from tok on, `left` of them
                    if (MORE && t0 + c < 2 * lead) {                  // eight tokens, two pieces each
#pragma unroll
                        for (int j = 0; j < 8; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) + __uint_as_float(r[j + 8]));
                        tok = (t0 + c) / 2;
                        left = 8;
                    }
                    if (kind == LIN_SWIGLU) {
                        // lanes 0-15 hold gates, 16-31 the ups of the same units: the lower half finishes even tokens, the upper half odd ones
                        const int unit = (r0 - sg.row0) / 2 + (lane & 15), hi = lane >> 4;
                        const LinActColumn to(sg, tok, unit, act);
#pragma unroll
                        for (int j = 0; j < 16; j += 2) {
                            const float give = __uint_as_float(hi ? r[j] : r[j + 1]), got = __shfl_xor_sync(~0u, give, 16);
                            const float gate = hi ? got : __uint_as_float(r[j]), up = hi ? __uint_as_float(r[j + 1]) : got;
                            if (j + hi < left && unit < sg.count) to.put(j + hi, lin_silu(gate) * up);
                        }
                    } else if (col < sg.count) {
                        if (kind == LIN_ADD) {
                            float *d = static_cast<float *>(sg.dst) + (size_t)tok * sg.ld + col;
                            float old[16];
#pragma unroll
                            for (int j = 0; j < 16; ++j) old[j] = j < left ? d[(size_t)j * sg.ld] : 0.f;
#pragma unroll
                            for (int j = 0; j < 16; ++j)
                                if (j < left) d[(size_t)j * sg.ld] = old[j] + __uint_as_float(r[j]);
                        } else if (kind == LIN_F32) {
                            float *d = static_cast<float *>(sg.dst) + (size_t)tok * sg.ld + col;
                            if (left >= 16) {
#pragma unroll
                                for (int j = 0; j < 16; ++j) d[(size_t)j * sg.ld] = __uint_as_float(r[j]);
                            } else {
#pragma unroll
                                for (int j = 0; j < 15; ++j)
                                    if (j < left) d[(size_t)j * sg.ld] = __uint_as_float(r[j]);
                            }
                        } else if (!MORE || kind == LIN_ACT) {
                            const LinActColumn to(sg, tok, col, act);
#pragma unroll
                            for (int j = 0; j < 16; ++j)
                                if (j < left) to.put(j, __uint_as_float(r[j]));
                        } else {
                            lin_store_column(segs, sg, tok, left, col, r);
                        }
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(tempty + (u & 1) * 8);
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (warp == 2) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(2 * tl.columns));
}

typedef CUresult (*lt_encode_fn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *, const cuuint32_t *,
                                 CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
// bfloat16 [rows][ld], `cols` of them in use: boxes of 64 columns x box_rows, 128-byte swizzle, zeros outside
static int lt_encode(CUtensorMap *map, const void *base, int cols, long long rows, long long ld, int box_rows)
{
    static lt_encode_fn fn = nullptr;
    if (!fn) {
        void *p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess)
            return ckb_fail(CKB_ERR_CUDA, "linear_tc: cuTensorMapEncodeTiled is not available");
        fn = (lt_encode_fn)p;
    }
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {LT_K, (cuuint32_t)box_rows}, estr[2] = {1, 1};
    if (fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
           CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
        return ckb_fail(CKB_ERR_SHAPE, "linear_tc: no tensor map for %lld x %d rows of %lld elements", rows, cols, ld);
    return 0;
}

template <int NT, bool MORE>
static int lt_launch(const LinMat *w, const void *x, int ldx, int tokens, int lead, int width, const LinSegs *segs, cudaStream_t st)
{
    static bool attr = false;
    if (!attr) {
        if (ckb_check_cuda((int)cudaFuncSetAttribute(linear_tc_kernel<NT, MORE>, cudaFuncAttributeMaxDynamicSharedMemorySize, LT_SMEM + LT_BARS + 1024), "linear_tc smem")) return CKB_ERR_CUDA;
        attr = true;
    }
    CUtensorMap wmap, xmap;
    static_assert(sizeof wmap == sizeof w->tmap, "tensor map size");
    memcpy(&wmap, w->tmap, sizeof wmap);
    const LtTile tile(width);
    int x0 = 0;
    for (int i = 0; i < segs->n; ++i) x0 = segs->s[i].x0 > x0 ? segs->s[i].x0 : x0;
    if (lt_encode(&xmap, x, x0 + w->cols, tokens + lead, ldx, width)) return CKB_ERR_SHAPE;
    const int tiles = (w->rows + LT_ROWS - 1) / LT_ROWS * ((tokens + lead + width - 1) / width);
    const int grid = tiles < ckb_sm_count() ? tiles : ckb_sm_count();
    return launch_pdl("linear_tc", linear_tc_kernel<NT, MORE>, dim3(grid), dim3(LT_THREADS), (size_t)tile.smem(), st, wmap, xmap, w->rows, w->cols / LT_K, tokens, lead, tile, *segs,
                      ckb_device_error_word());
}
template <bool MORE>
static int lt_pick(const LinMat *w, const void *x, int ldx, int tokens, int lead, int width, const LinSegs *segs, cudaStream_t st)
{
    switch (width) {
        case 32: return lt_launch<32, MORE>(w, x, ldx, tokens, lead, width, segs, st);
        case 64: return lt_launch<64, MORE>(w, x, ldx, tokens, lead, width, segs, st);
        case 128: return lt_launch<128, MORE>(w, x, ldx, tokens, lead, width, segs, st);
        case 256: return lt_launch<256, MORE>(w, x, ldx, tokens, lead, width, segs, st);
        default: return lt_launch<0, MORE>(w, x, ldx, tokens, lead, width, segs, st);
    }
}

}  // namespace ckb

using namespace ckb;

extern "C" int ckb_linear_encode(LinMat *w)
{
    CUtensorMap m;
    if (lt_encode(&m, w->w, w->cols, w->rows, w->cols, LT_ROWS)) return CKB_ERR_SHAPE;
    memcpy(w->tmap, &m, sizeof m);
    return 0;
}

extern "C" int ckb_launch_linear_tc(const LinMat *w, const void *x, int ldx, int tokens, const LinSegs *segs, void *stream)
{
    const int lead = segs->act < 0 ? -segs->act : 0;
    if (w->rows % 32 || w->cols % LT_K || ldx % 8 || ((uintptr_t)x & 15)) return ckb_fail(CKB_ERR_ALIGN, "linear_tc: %d x %d, rows of %d", w->rows, w->cols, ldx);
    if (segs->act == ACT_F32 || lead % 8 || lead > tokens) return ckb_fail(CKB_ERR_SHAPE, "linear_tc: activation type %d for %d rows", segs->act, tokens);
    bool more = lead > 0;
    for (int i = 0; i < segs->n; ++i) {
        if (segs->s[i].x0 % LT_K || (segs->s[i].x0 != (i ? segs->s[i - 1].x0 : 0) && segs->s[i].row0 % LIN_INPUT_ROWS)) return ckb_fail(CKB_ERR_ALIGN, "linear_tc: input of segment %d", i);
        more = more || segs->s[i].kind >= LIN_SILU || segs->s[i].x0;
    }
    // token tile: fewest rounds over the SMs, each round as long as its tile is wide (plus what a tile costs whatever its width).  Narrow
    // tiles are bound by the loading and issuing threads' own instructions: only widths that are known at compile time
    const int sms = ckb_sm_count(), rt = (w->rows + LT_ROWS - 1) / LT_ROWS, in_rows = tokens + lead;
    int best = 0;
    long long best_cost = 0;
    for (int n = LT_MAX_WIDTH; n >= 32; n = n > 128 ? n - 16 : n / 2) {
        const int tt = (in_rows + n - 1) / n;
        if (n > 32 && tt == 1 && (n > 128 ? n - 16 : n / 2) >= in_rows) continue;
        const long long rounds = ((long long)rt * tt + sms - 1) / sms, cost = rounds * (n + 48);
        if (!best || cost < best_cost) { best = n; best_cost = cost; }
    }
    cudaStream_t st = ckb_stream(stream);
    return more ? lt_pick<true>(w, x, ldx, tokens, lead, best, segs, st) : lt_pick<false>(w, x, ldx, tokens, lead, best, segs, st);
}
