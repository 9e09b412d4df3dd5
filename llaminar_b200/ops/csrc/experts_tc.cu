// Products of rows that are sorted by expert, on the 5th-generation tensor cores: tiles of 128 rows of one expert x 256 weight rows.
//
// Persistent CTAs walk the tiles (columns fastest, so that the CTAs at work share row and weight tiles in L2).  Row and weight tiles of
// 64 columns arrive by TMA, 128-byte swizzled; one MMA of M = 128, N = 256 per 16 columns; two accumulators of 256 columns in TMEM, so
// that the epilogue of a tile runs under the products of the next.  PAIR: the 256 weight rows are 128 rows of the gate and the 128 of
// `up` at the same place, and the epilogue writes silu(gate) * up, or its limited form.  A row tile may reach into the next expert's rows: they are not stored.
// Warp 0 TMA, 1 MMA issue and TMEM allocation, 2 to 5 epilogue.  Every wait is bounded; on a timeout the status word is raised.
#include "experts.h"
#include "launch.h"
#include "tc_tile.cuh"

namespace llm {
namespace etc {
using namespace tc5;

constexpr int THREADS = 192, BM = 128, BN = 256, STAGES = 4, STAGE = 3 * ATOM;      // a stage: one atom of rows, two of weights
constexpr size_t SMEM = (size_t)STAGES * STAGE + 1024;
enum Bar { FULL = 0, EMPTY = FULL + STAGES, T_FULL = EMPTY + STAGES, T_EMPTY = T_FULL + 2, N_BARS = T_EMPTY + 2 };

struct Tile { int expert, row0, rows, n0; };

template <bool PAIR>
__global__ void __launch_bounds__(THREADS, 1) expert_grouped_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w,
                                                                    const ExpertGroupedParams p, int* status) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t s_bars[N_BARS];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort[2];
    __shared__ int s_row[EXPERTS_MAX + 1], s_tile[EXPERTS_MAX + 1];         // first row and first row tile of every expert
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u, bars = smem_u32(s_bars);
    auto bar = [&](int i) { return bars + i * 8; };
    if (tid == 0) {
        s_abort[0] = 0; s_abort[1] = 0;
        for (int i = 0; i < N_BARS; ++i) mbar_init(bar(i), i >= T_EMPTY ? 4 : 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        fence_proxy_async();
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    pdl_wait();
    if (warp == 0) {                               // running sums of rows and tiles
        int rows = 0, tiles = 0;
        for (int e0 = 0; e0 < p.experts; e0 += 32) {
            const int c = e0 + lane < p.experts ? p.counts[e0 + lane] : 0;
            int r = c, t = (c + BM - 1) / BM;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int a = __shfl_up_sync(0xffffffffu, r, o), b = __shfl_up_sync(0xffffffffu, t, o);
                if (lane >= o) { r += a; t += b; }
            }
            if (e0 + lane < p.experts) { s_row[e0 + lane + 1] = rows + r; s_tile[e0 + lane + 1] = tiles + t; }
            rows += __shfl_sync(0xffffffffu, r, 31);
            tiles += __shfl_sync(0xffffffffu, t, 31);
        }
        if (lane == 0) s_row[0] = s_tile[0] = 0;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    volatile int* abort_flag = s_abort;
    constexpr int COLS = PAIR ? BN / 2 : BN;       // columns of the result per tile
    const int n_cols = (p.n + COLS - 1) / COLS, total = s_tile[p.experts] * n_cols, steps = (p.k + 63) / 64;
    auto tile_of = [&](int i) {
        const int rt = i / n_cols;
        int lo = 0, hi = p.experts - 1;            // the expert whose tiles hold rt
        while (lo < hi) {
            const int mid = (lo + hi + 1) / 2;
            if (s_tile[mid] <= rt) lo = mid; else hi = mid - 1;
        }
        Tile t;
        t.expert = lo;
        t.row0 = s_row[lo] + (rt - s_tile[lo]) * BM;
        t.rows = min(BM, s_row[lo + 1] - t.row0);
        t.n0 = (i - rt * n_cols) * COLS;
        return t;
    };

    if (warp == 0) {
        if (elect_one()) {
            bool ok = true;
            int s = 0, phase = 1;
            for (int i = blockIdx.x; i < total && ok; i += gridDim.x) {
                const Tile t = tile_of(i);
                for (int k = 0; k < steps; ++k) {
                    ok = mbar_wait(bar(EMPTY + s), phase, abort_flag);
                    if (!ok) break;
                    const uint32_t dst = base + s * STAGE;
                    mbar_arrive_expect_tx(bar(FULL + s), STAGE);
                    tma_load_2d(dst, &map_x, k * 64, t.row0, bar(FULL + s));
                    tma_load_3d(dst + ATOM, &map_w, k * 64, t.n0, t.expert, bar(FULL + s));
                    tma_load_3d(dst + 2 * ATOM, &map_w, k * 64, PAIR ? p.n + t.n0 : t.n0 + BN / 2, t.expert, bar(FULL + s));
                    if (++s == STAGES) { s = 0; phase ^= 1; }
                }
            }
        }
    } else if (warp == 1) {
        constexpr uint32_t idesc = instr_desc(BN);
        bool ok = true;
        int s = 0, phase = 0, n = 0;
        for (int i = blockIdx.x; i < total && ok; i += gridDim.x, ++n) {
            const int b = n & 1;
            ok = mbar_wait_warp(bar(T_EMPTY + b), ((n >> 1) & 1) ^ 1, abort_flag);
            if (!ok) break;
            tc_fence_after();
            for (int k = 0; k < steps; ++k) {
                ok = mbar_wait_warp(bar(FULL + s), phase, abort_flag);
                if (!ok) break;
                tc_fence_after();
                if (elect_one()) {
                    const uint64_t a = smem_desc_sw128(base + s * STAGE), w = smem_desc_sw128(base + s * STAGE + ATOM);
                    const int ks = min(4, (p.k - k * 64 + 15) / 16);       // columns past the end are zeros
                    for (int j = 0; j < ks; ++j) mma_f16(tmem + b * BN, a + 2 * j, w + 2 * j, idesc, k + j > 0 ? 1u : 0u);
                    mma_commit(bar(EMPTY + s));
                    if (k + 1 == steps) mma_commit(bar(T_FULL + b));
                }
                __syncwarp();
                if (++s == STAGES) { s = 0; phase ^= 1; }
            }
        }
    } else {
        const int q4 = warp & 3, row = q4 * 32 + lane;         // a warp reads its quarter of the TMEM lanes
        const uint32_t t_lane = tmem + ((uint32_t)(q4 * 32) << 16);
        bool ok = true;
        int n = 0;
        for (int i = blockIdx.x; i < total && ok; i += gridDim.x, ++n) {
            const int b = n & 1;
            const Tile t = tile_of(i);
            ok = mbar_wait_warp(bar(T_FULL + b), (n >> 1) & 1, abort_flag);
            if (!ok) break;
            tc_fence_after();
            const uint32_t acc = t_lane + b * BN;
            __nv_bfloat16* out = p.out + (size_t)(t.row0 + row) * p.n + t.n0;
#pragma unroll 1
            for (int c = 0; c < COLS; c += 32) {
                if (t.n0 + c >= p.n) break;                    // the same for the warp
                uint32_t r[32], u[32];
                tmem_ld32_issue(acc + c, r);
                if constexpr (PAIR) tmem_ld32_issue(acc + BN / 2 + c, u);
                tmem_wait_ld(r);
                if constexpr (PAIR) {
                    tmem_wait_ld(u);
#pragma unroll
                    for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(expert_pair(__uint_as_float(r[j]), __uint_as_float(u[j]), p.limit));
                }
                if (row < t.rows) {
#pragma unroll
                    for (int j = 0; j < 32; j += 8) {
                        if (t.n0 + c + j >= p.n) break;        // p.n is a multiple of 8
                        uint32_t w[4];
#pragma unroll
                        for (int x = 0; x < 4; ++x) w[x] = pack_bf16(__uint_as_float(r[j + 2 * x]), __uint_as_float(r[j + 2 * x + 1]));
                        *reinterpret_cast<uint4*>(out + c + j) = make_uint4(w[0], w[1], w[2], w[3]);
                    }
                }
                __syncwarp();
            }
            tc_fence_before();
            __syncwarp();
            mbar_arrive_if(bar(T_EMPTY + b), lane == 0);
        }
    }
    tc_fence_before();
    __syncthreads();
    teardown(abort_flag, tid, status);
    if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512) : "memory");
}

}  // namespace etc

bool expert_grouped_fits(int n, int k, int experts) { return n >= 8 && k >= 8 && n % 8 == 0 && k % 8 == 0 && experts <= EXPERTS_MAX; }

cudaError_t launch_expert_grouped(const __nv_bfloat16* w, const __nv_bfloat16* x, const ExpertGroupedParams& p, bool pair_act, int* status, cudaStream_t st) {
    using namespace etc;
    if (p.pairs == 0) return cudaSuccess;
    if (!expert_grouped_fits(p.n, p.k, p.experts)) return cudaErrorInvalidValue;
    const cuuint64_t rows = (cuuint64_t)p.n * (pair_act ? 2 : 1);
    CUtensorMap mx, mw;
    if (!make_map(&mx, x, p.k, p.pairs, p.k, BM) ||
        !make_map_nd<3>(&mw, w, {(cuuint64_t)p.k, rows, (cuuint64_t)p.experts}, {(cuuint64_t)p.k, rows * p.k}, {64, BN / 2, 1}))
        return cudaErrorInvalidValue;
    static int sms = 0;
    if (!sms) {
        int dev = 0;
        cudaGetDevice(&dev);
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    }
    const int cols = pair_act ? BN / 2 : BN, most = (p.pairs / BM + min(p.experts, p.pairs)) * ((p.n + cols - 1) / cols);
    auto go = [&](auto kernel) {
        cudaError_t e = raise_smem(kernel, SMEM);
        return e != cudaSuccess ? e : launch_pdl(kernel, dim3(min(sms, most)), dim3(THREADS), SMEM, st, mx, mw, p, status);
    };
    return pair_act ? go(expert_grouped_kernel<true>) : go(expert_grouped_kernel<false>);
}

}  // namespace llm
