// Mixture-of-experts feed-forwards with unquantised matrices: routing, sorting by expert, and the products of few rows.
#include <cooperative_groups.h>

#include "common.cuh"
#include "experts.h"
#include "launch.h"

namespace llm {

namespace {

namespace cg = cooperative_groups;

LLM_DEVICE float to_f(float v) { return v; }
LLM_DEVICE float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <class T> LLM_DEVICE T from_f(float v);
template <> LLM_DEVICE float from_f<float>(float v) { return v; }
template <> LLM_DEVICE __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

LLM_DEVICE void unpack8(const uint4& w, float (&v)[8]) {
    const uint32_t x[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) { v[2 * j] = bf16_lo(x[j]); v[2 * j + 1] = bf16_hi(x[j]); }
}
LLM_DEVICE void load8(const __nv_bfloat16* p, float (&v)[8]) { unpack8(*reinterpret_cast<const uint4*>(p), v); }
LLM_DEVICE void load8(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}

// ---- routing -------------------------------------------------------------------------------------------------------------------
// A warp's view of which groups of experts may be chosen: up to 32 groups as a bit mask, more in shared memory.
struct Groups {
    unsigned mask;                                 // of the groups that stay
    const unsigned* g;                             // zero where a group stays; nullptr: the mask holds
    int size;                                      // experts of a group (0: all may be chosen)
    LLM_DEVICE bool stays(int i) const { return size == 0 || (g ? g[i / size] == 0 : (mask >> (i / size)) & 1u); }
};

// One warp: marks the `keep` groups of neighbours with the largest values in z[0 .. n) by a zero in g[0 .. groups).
LLM_DEVICE unsigned ordered(float v) {             // integers of the same order; 0 is below all of them
    const unsigned u = __float_as_uint(v);
    return u & 0x80000000u ? ~u : u | 0x80000000u;
}
LLM_DEVICE Groups keep_groups(const float* z, unsigned* g, const ExpertRouteParams& p) {
    const int lane = threadIdx.x & 31, size = p.n / p.groups;
    if (p.groups <= 32) {                          // a group per lane: it stays if fewer than `keep` are ahead of it
        unsigned best = 0;
        if (lane < p.groups) for (int j = 0; j < size; ++j) best = max(best, ordered(z[lane * size + j]));
        int ahead = 0;
        for (int j = 0; j < p.groups; ++j) {
            const unsigned other = __shfl_sync(0xffffffffu, best, j);
            ahead += other > best || (other == best && j < lane);
        }
        return {__ballot_sync(0xffffffffu, lane < p.groups && ahead < p.keep), nullptr, size};
    }
    for (int i = lane; i < p.groups; i += 32) {
        unsigned best = 1;
        for (int j = 0; j < size; ++j) best = max(best, ordered(z[i * size + j]));
        g[i] = best;
    }
    __syncwarp();
    for (int r = 0; r < p.keep; ++r) {
        unsigned best = 0, at = 0xffffffffu;
        for (int i = lane; i < p.groups; i += 32)
            if (g[i] > best) { best = g[i]; at = i; }
        const unsigned top = __reduce_max_sync(0xffffffffu, best);
        at = __reduce_min_sync(0xffffffffu, best == top ? at : 0xffffffffu);
        if (lane == 0 && at < (unsigned)p.groups) g[at] = 0;
        __syncwarp();
    }
    return {0u, g, size};
}

// One warp: the `top` largest of z[0 .. n), of the groups that stay, and the softmax over them.  Logits stay in registers as integers of the same order (NR per
// lane), so a round is two warp-wide integer reductions.  Every id it writes is a valid expert, whatever the logits are.
template <int NR>
LLM_DEVICE void choose_of(const float* z, const Groups& groups, const ExpertRouteParams& p, int t) {
    const int lane = threadIdx.x & 31;
    unsigned key[NR];
#pragma unroll
    for (int j = 0; j < NR; ++j) {
        const int i = lane + j * 32;
        key[j] = i < p.n && groups.stays(i) ? ordered(z[i]) : 0u;
    }
    float mine = -INFINITY;                        // lane r: the r-th largest logit
    int id = 0;
    for (int r = 0; r < p.top; ++r) {
        unsigned best = 0;
#pragma unroll
        for (int j = 0; j < NR; ++j) best = max(best, key[j]);
        best = __reduce_max_sync(0xffffffffu, best);
        unsigned at = 0xffffffffu;                 // the lowest expert that has it
#pragma unroll
        for (int j = 0; j < NR; ++j)
            if (key[j] == best && lane + j * 32 < p.n) at = min(at, (unsigned)(lane + j * 32));
        at = __reduce_min_sync(0xffffffffu, at);
#pragma unroll
        for (int j = 0; j < NR; ++j)
            if ((unsigned)(lane + j * 32) == at) key[j] = 0;
        if (lane == r) { mine = z[at]; id = at; }
    }
    const float top = warp_max(mine), e = lane < p.top ? expf(mine - top) : 0.f, sum = warp_sum(e);      // every lane takes part
    if (lane < p.top) {
        const size_t pair = (size_t)t * p.top + lane;
        p.ids[pair] = id;
        p.weights[pair] = e / sum;
        if (p.counts) p.ranks[pair] = atomicAdd(&p.counts[id], 1);
    }
}
LLM_DEVICE void choose(const float* z, unsigned* g, const ExpertRouteParams& p, int t) {       // g: workspace for the groups
    const Groups groups = p.keep < p.groups ? keep_groups(z, g, p) : Groups{0u, nullptr, 0};
    if (p.n <= 32) choose_of<1>(z, groups, p, t);
    else if (p.n <= 128) choose_of<4>(z, groups, p, t);
    else choose_of<EXPERTS_MAX / 32>(z, groups, p, t);
}

// A cluster of CTAs per token: their warps take the experts in turn, four at a time, and leave the logits with the first CTA.
constexpr int ROUTE_THREADS = 512, ROUTE_CLUSTER = 8;
template <class T, bool VEC>
__global__ void __launch_bounds__(ROUTE_THREADS) expert_route_kernel(const ExpertRouteParams p) {
    __shared__ float z[EXPERTS_MAX];
    __shared__ unsigned s_groups[EXPERTS_MAX];
    pdl_trigger();
    cg::cluster_group cluster = cg::this_cluster();
    const bool spread = gridDim.x > 1;
    if (spread) cluster.sync();                    // every CTA runs: its memory may be written
    pdl_wait();
    const int t = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    constexpr int WARPS = ROUTE_THREADS / 32, NE = 4;
    float* dst = spread ? cluster.map_shared_rank(z, 0) : z;
    const T* x = static_cast<const T*>(p.x) + (size_t)t * p.x_row;
    for (int e0 = (warp * gridDim.x + blockIdx.x) * NE; e0 < p.n; e0 += WARPS * NE * gridDim.x) {
        float acc[NE] = {};
        const T* w[NE];
#pragma unroll
        for (int j = 0; j < NE; ++j) w[j] = static_cast<const T*>(p.router) + (size_t)min(e0 + j, p.n - 1) * p.d;
        if constexpr (VEC) {
#pragma unroll 2
            for (int c = lane * 8; c < p.d; c += 256) {
                float a[8], b[NE][8];
                load8(x + c, a);
#pragma unroll
                for (int j = 0; j < NE; ++j) load8(w[j] + c, b[j]);
#pragma unroll
                for (int j = 0; j < NE; ++j)
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[j] = fmaf(a[i], b[j][i], acc[j]);
            }
        } else {
            for (int c = lane; c < p.d; c += 32)
#pragma unroll
                for (int j = 0; j < NE; ++j) acc[j] = fmaf(to_f(x[c]), to_f(w[j][c]), acc[j]);
        }
#pragma unroll
        for (int j = 0; j < NE; ++j) {
            const float s = warp_sum(acc[j]);
            if (lane == 0 && e0 + j < p.n) dst[e0 + j] = p.bias ? s + p.bias[e0 + j] : s;
        }
    }
    if (spread) cluster.sync(); else __syncthreads();
    if (warp == 0 && blockIdx.x == 0) choose(z, s_groups, p, t);
}

// a warp per token, logits given
__global__ void __launch_bounds__(128) expert_choose_kernel(const ExpertRouteParams p, int rows) {
    extern __shared__ float sm[];
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x * 4 + warp;
    if (t >= rows) return;
    float* z = sm + warp * (p.n + p.groups);
    for (int i = lane; i < p.n; i += 32) z[i] = p.logits[(size_t)t * p.n + i] + (p.bias ? p.bias[i] : 0.f);
    __syncwarp();
    choose(z, reinterpret_cast<unsigned*>(z + p.n), p, t);
}

// a CTA per token; warp j finds the row of the token's pair j, then all threads copy
__global__ void __launch_bounds__(256) expert_place_kernel(const ExpertPlaceParams p) {
    __shared__ int s_row[EXPERTS_MAX_TOP];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int j = warp; j < p.top; j += 8) {
        const int pair = t * p.top + j, e = LLM_CHECK_INDEX(p.ids[pair], p.n);
        int before = 0;
        for (int i = lane; i < e; i += 32) before += p.counts[i];
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
        if (lane == 0) p.place[pair] = s_row[j] = before + p.ranks[pair];
    }
    __syncthreads();
    const uint4* src = reinterpret_cast<const uint4*>(p.x + (size_t)t * p.x_row);
    for (int u = threadIdx.x; u < p.d / 8; u += 256) {
        const uint4 v = src[u];
        for (int j = 0; j < p.top; ++j) reinterpret_cast<uint4*>(p.xs + (size_t)s_row[j] * p.d)[u] = v;
    }
}

// ---- few pairs -------------------------------------------------------------------------------------------------------------------
// As the small-batch product of dense matrices (gemv_dense): weights are the M operand, 16 rows per warp, pairs the N operand, eight
// per MMA; both operands use the same permutation of k, so every fragment is a plain 16-byte load.  `wk` warps share the K range of a
// row block.  A CTA serves one expert: blockIdx.y names it, or (by_pair, fewer pairs than experts) a pair, whose CTA stands for its
// expert if no earlier pair has the same.
constexpr int ROW_WARPS = 8;
LLM_DEVICE void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <bool PAIR, int NG>                       // NG: groups of eight pairs per pass over the weights
__global__ void __launch_bounds__(32 * ROW_WARPS) expert_rows_kernel(const ExpertRowsParams p, int wk, bool by_pair) {
    constexpr int NA = PAIR ? 2 : 1, NW = 2 * NA, UN = PAIR ? 4 : 8;
    __shared__ float s_acc[ROW_WARPS][NA][16][9];
    __shared__ short s_pair[EXPERT_ROWS_MAX_PAIRS];
    __shared__ int s_count;
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int e = by_pair ? LLM_CHECK_INDEX(p.ids[blockIdx.y], p.experts) : (int)blockIdx.y;
    if (warp == 0) {
        int n = 0;
#pragma unroll 4
        for (int i0 = 0; i0 < p.pairs; i0 += 32) {
            const int i = i0 + lane;
            const bool hit = i < p.pairs && p.ids[i] == e;
            const unsigned m = __ballot_sync(0xffffffffu, hit);
            if (hit) s_pair[n + __popc(m & ((1u << lane) - 1))] = (short)i;
            n += __popc(m);
        }
        if (lane == 0) s_count = n;
    }
    __syncthreads();
    const int count = s_count;
    if (count == 0 || (by_pair && s_pair[0] != (int)blockIdx.y)) return;
    const int part = warp % wk, n0 = (blockIdx.x * (ROW_WARPS / wk) + warp / wk) * 16;
    const int blocks = (p.k + 31) / 32, per = (blocks + wk - 1) / wk, kb0 = part * per, kb1 = min(blocks, kb0 + per);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    const __nv_bfloat16* w[NW];                    // rows past the end repeat the last one (never stored)
#pragma unroll
    for (int i = 0; i < NW; ++i)
        w[i] = static_cast<const __nv_bfloat16*>(p.w) + ((size_t)e * NA * p.n + min(n0 + g + (i & 1) * 8, p.n - 1) + (size_t)(i >> 1) * p.n) * p.k + t * 8;
    const bool live = n0 < p.n;
    for (int q0 = 0; q0 < count; q0 += 8 * NG) {
        float acc[NG][NA][4] = {};
        const __nv_bfloat16* x[NG];
#pragma unroll
        for (int q = 0; q < NG; ++q)
            x[q] = static_cast<const __nv_bfloat16*>(p.x) + (size_t)(s_pair[min(q0 + q * 8 + g, count - 1)] / p.div) * p.x_row + t * 8;
        for (int kb = kb0; kb < kb1 && live; kb += UN) {
            uint4 wv[UN][NW];
#pragma unroll
            for (int u = 0; u < UN; ++u) {
                const bool in = kb + u < kb1 && (kb + u) * 32 + t * 8 < p.k;
#pragma unroll
                for (int i = 0; i < NW; ++i) wv[u][i] = in ? ldg_nc_v4(w[i] + (size_t)(kb + u) * 32) : zero;
            }
#pragma unroll
            for (int q = 0; q < NG; ++q) {
                if (q0 + q * 8 >= count) break;
                uint4 xv[UN];
#pragma unroll
                for (int u = 0; u < UN; ++u) {
                    const bool in = kb + u < kb1 && (kb + u) * 32 + t * 8 < p.k;
                    xv[u] = in ? *reinterpret_cast<const uint4*>(x[q] + (size_t)(kb + u) * 32) : zero;
                }
#pragma unroll
                for (int u = 0; u < UN; ++u)
#pragma unroll
                    for (int i = 0; i < NA; ++i) {
                        mma_bf16(acc[q][i], wv[u][2 * i].x, wv[u][2 * i + 1].x, wv[u][2 * i].y, wv[u][2 * i + 1].y, xv[u].x, xv[u].y);
                        mma_bf16(acc[q][i], wv[u][2 * i].z, wv[u][2 * i + 1].z, wv[u][2 * i].w, wv[u][2 * i + 1].w, xv[u].z, xv[u].w);
                    }
            }
        }
        const int rb = ROW_WARPS / wk;
#pragma unroll
        for (int q = 0; q < NG; ++q) {
            const int m = min(8, count - q0 - q * 8);
            if (m <= 0) break;                     // the same for all threads
            __syncthreads();
#pragma unroll
            for (int i = 0; i < NA; ++i) {
                s_acc[warp][i][g][2 * t] = acc[q][i][0]; s_acc[warp][i][g][2 * t + 1] = acc[q][i][1];
                s_acc[warp][i][g + 8][2 * t] = acc[q][i][2]; s_acc[warp][i][g + 8][2 * t + 1] = acc[q][i][3];
            }
            __syncthreads();
            for (int i = threadIdx.x; i < rb * 16 * m; i += 32 * ROW_WARPS) {
                const int c = i % (rb * 16), r = i / (rb * 16), n = blockIdx.x * rb * 16 + c;
                if (n >= p.n) continue;
                float v = 0.f, v2 = 0.f;
                for (int a = 0; a < wk; ++a) {
                    v += s_acc[(c / 16) * wk + a][0][c % 16][r];
                    if constexpr (PAIR) v2 += s_acc[(c / 16) * wk + a][1][c % 16][r];
                }
                if constexpr (PAIR) v = expert_pair(v, v2, p.limit);
                static_cast<__nv_bfloat16*>(p.out)[(size_t)s_pair[q0 + q * 8 + r] * p.n + n] = __float2bfloat16(v);
            }
        }
    }
}

// ---- any size, float arithmetic: a warp per pair and output value ----------------------------------------------------------------
template <class T, bool PAIR>
__global__ void __launch_bounds__(256) expert_plain_kernel(const ExpertRowsParams p) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, pair = blockIdx.x, e = LLM_CHECK_INDEX(p.ids[pair], p.experts);
    const T* x = static_cast<const T*>(p.x) + (size_t)(pair / p.div) * p.x_row;
    const T* w = static_cast<const T*>(p.w) + (size_t)e * (PAIR ? 2 : 1) * p.n * p.k;
    for (int n = blockIdx.y * 8 + (threadIdx.x >> 5); n < p.n; n += gridDim.y * 8) {
        float a = 0.f, b = 0.f;
        for (int c = lane; c < p.k; c += 32) {
            const float v = to_f(x[c]);
            a = fmaf(v, to_f(w[(size_t)n * p.k + c]), a);
            if (PAIR) b = fmaf(v, to_f(w[((size_t)p.n + n) * p.k + c]), b);
        }
        a = warp_sum(a);
        if (PAIR) { b = warp_sum(b); a = p.limit > 0.f ? limited_pair(a, b, p.limit, [](float z) { return 1.f / (1.f + expf(-z)); }) : a / (1.f + expf(-a)) * b; }
        if (lane == 0) static_cast<T*>(p.out)[(size_t)pair * p.n + n] = from_f<T>(a);
    }
}

}  // namespace

cudaError_t launch_expert_route(const ExpertRouteParams& p, int rows, bool f32, cudaStream_t st) {
    if (rows == 0) return cudaSuccess;
    if (p.n < 1 || p.n > EXPERTS_MAX || p.top < 1 || p.top > p.n || p.top > EXPERTS_MAX_TOP) return cudaErrorInvalidValue;
    if (p.groups < 1 || p.n % p.groups || p.keep < 1 || p.keep > p.groups || p.top > p.n / p.groups * p.keep) return cudaErrorInvalidValue;
    if (p.logits) return launch_pdl(expert_choose_kernel, dim3((rows + 3) / 4), dim3(128), (size_t)4 * (p.n + p.groups) * 4, st, p, rows);
    const bool vec = p.d % 8 == 0 && p.x_row % 8 == 0 && !((reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.router)) & 15);
    if (rows > 65535) return cudaErrorInvalidValue;
    auto go = [&](auto kernel) {
        cudaLaunchConfig_t cfg = {};
        const int ctas = rows <= 16 && p.n >= 32 ? ROUTE_CLUSTER : 1;      // few tokens: the router's rows are read by more SMs
        cfg.gridDim = dim3(ctas, rows);
        cfg.blockDim = dim3(ROUTE_THREADS);
        cfg.stream = st;
        cudaLaunchAttribute attr[2];
        attr[0].id = cudaLaunchAttributeClusterDimension;
        attr[0].val.clusterDim.x = ctas; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
        attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[1].val.programmaticStreamSerializationAllowed = 1;
        cfg.attrs = attr;
        cfg.numAttrs = pdl_enabled() ? 2 : 1;
        return cudaLaunchKernelEx(&cfg, kernel, p);
    };
    if (f32) return vec ? go(expert_route_kernel<float, true>) : go(expert_route_kernel<float, false>);
    return vec ? go(expert_route_kernel<__nv_bfloat16, true>) : go(expert_route_kernel<__nv_bfloat16, false>);
}

cudaError_t launch_expert_place(const ExpertPlaceParams& p, int rows, cudaStream_t st) {
    if (rows == 0) return cudaSuccess;
    if (p.d % 8 || p.x_row % 8 || p.top > EXPERTS_MAX_TOP) return cudaErrorInvalidValue;
    return launch_pdl(expert_place_kernel, dim3(rows), dim3(256), 0, st, p);
}

cudaError_t launch_expert_rows(const ExpertRowsParams& p, cudaStream_t st) {
    if (p.pairs == 0) return cudaSuccess;
    if (p.pairs > EXPERT_ROWS_MAX_PAIRS || p.k % 8 || p.x_row % 8 || p.n < 1 || p.div < 1) return cudaErrorInvalidValue;
    const bool by_pair = p.pairs < p.experts;
    const int active = by_pair ? p.pairs : p.experts;
    const int blocks = (p.k + 31) / 32, tiles = (p.n + 15) / 16 * active;
    int wk = 1;                                    // split K until every warp has about eight blocks of 32 and the grid fills the machine
    while (wk < ROW_WARPS && blocks >= 16 * wk && (blocks > 64 * wk || tiles * wk < 148 * 32)) wk *= 2;
    const int cols = ROW_WARPS / wk * 16;
    const dim3 grid((p.n + cols - 1) / cols, active);
    auto go = [&](auto kernel) { return launch_pdl(kernel, grid, dim3(32 * ROW_WARPS), 0, st, p, wk, by_pair); };
    const int each = p.pairs / p.experts;          // pairs of an expert, on average
    if (p.pair_act) return each >= 12 ? go(expert_rows_kernel<true, 4>) : each >= 4 ? go(expert_rows_kernel<true, 2>) : go(expert_rows_kernel<true, 1>);
    return each >= 12 ? go(expert_rows_kernel<false, 4>) : each >= 4 ? go(expert_rows_kernel<false, 2>) : go(expert_rows_kernel<false, 1>);
}

cudaError_t launch_expert_plain(const ExpertRowsParams& p, bool f32, cudaStream_t st) {
    if (p.pairs == 0) return cudaSuccess;
    const dim3 grid(p.pairs, min((p.n + 7) / 8, 65535));
    auto go = [&](auto kernel) { return launch_pdl(kernel, grid, dim3(256), 0, st, p); };
    if (f32) return p.pair_act ? go(expert_plain_kernel<float, true>) : go(expert_plain_kernel<float, false>);
    return p.pair_act ? go(expert_plain_kernel<__nv_bfloat16, true>) : go(expert_plain_kernel<__nv_bfloat16, false>);
}

LLM_DEFINE_BOUNDS_STATUS_READER(bounds_status_experts)

}  // namespace llm
