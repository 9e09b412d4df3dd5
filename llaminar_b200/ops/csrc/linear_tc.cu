// Linear attention over prompts on the 5th-generation tensor cores: mLSTM and retention, chunk-parallel.
//
// A sequence is cut into chunks of 128 rows.  With G_t the running sum of the log forget gates inside a chunk (retention: (t + 1) log
// decay), i_t the log input gates (retention: 0), a_j = i_j - G_j and A_t the running maximum of a, row t of a chunk whose state is S
// with stabiliser m has
//
//     o_t = sum_{j<=t} (q_t.k_j) e^(a_j - M_t) v_j + e^(m - M_t) S q_t        M_t = max(m, A_t)
//     normaliser max(|the same sum without v|, e^-(G_t + M_t))                (mLSTM)
//
// and the state behind a chunk of L rows is e^(m - M) S + e^(A_L - M) sum_j e^(a_j - A_L) v_j k_j^T with M = max(m, A_L), its
// stabiliser G_L + M.  Every exponent is <= 0.  (Retention: M_t = A_t, and S is scaled by e^(G_t).)  Three launches:
//
//   chunk_state   per chunk and head: sum_j e^(a_j - A_L) v_j k_j^T           tcgen05, M = 128 values, N = dim, K = 128 rows
//   chunk_scan    per head: the states in front of every chunk, one after the other, and the sequence's new state
//   chunk_out     per chunk and head: scores, weights, o, norm and gate      tcgen05, M = 128 rows, N = 128 rows / values
//
// What enters the state, the state and the weights stay at 32-bit accuracy: such operands are split into two bf16 numbers and
// multiplied twice (q, k and v as projected are bf16 already).  Logarithms are to base 2 inside the kernels.
// Every mbarrier wait is bounded; on a timeout the kernel raises the status word and tears down.
#include "launch.h"
#include "mixers.h"
#include "tc_tile.cuh"

namespace llm {
namespace lin {
using namespace tc5;

constexpr int C = LINEAR_CHUNK, THREADS = 256, VS = 128;        // VS: values (rows of the state) per CTA
constexpr float NORM_FLOOR = 1e-6f;

LLM_DEVICE float log2_decay(float d) { return d > 0.f ? log2f(d) : -1e30f; }
LLM_DEVICE void lstm_gates2(float zi, float zf, float cap, float& i, float& f) {      // log2 of input and forget gate
    i = cap * tanhf(zi / cap) * LOG2E;
    const float z = cap * tanhf(zf / cap);
    f = (z >= 0.f ? -log1pf(expf(-z)) : z - log1pf(expf(z))) * LOG2E;
}

// The chunk's a_j, G_t and A_t (see above), for the first 128 threads; every thread calls it.  Rows past `len`: a = -inf.
struct Gates { float a, g, top; };
LLM_DEVICE Gates retention_gates(float decay, int t) {
    const float g = (float)(t + 1) * log2_decay(decay);
    return {-g, g, -g};
}
LLM_DEVICE Gates chunk_gates(const LinearParams& p, int h, int r0, int len, float (&s_tmp)[2][4]) {
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5;
    Gates r = {-INFINITY, 0.f, -INFINITY};
    if (!p.gates) {
        if (t < len) r = retention_gates(p.decay[h], t);
        return r;
    }
    float i = -INFINITY, f = 0.f;
    if (t < len) {
        const float* z = p.gates + (size_t)(r0 + t) * p.gate_row;
        lstm_gates2(z[h] + p.bias_i[h], z[p.heads + h] + p.bias_f[h], p.cap, i, f);
    }
    if (t < C) {
        float s = f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, s, o); if (lane >= o) s += x; }
        if (lane == 31) s_tmp[0][warp] = s;
        r.g = s;
    }
    __syncthreads();
    if (t < C) {
        for (int w = 0; w < warp; ++w) r.g += s_tmp[0][w];
        r.a = i - r.g;
        float m = r.a;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, m, o); if (lane >= o) m = fmaxf(m, x); }
        if (lane == 31) s_tmp[1][warp] = m;
        r.top = m;
    }
    __syncthreads();
    if (t < C)
        for (int w = 0; w < warp; ++w) r.top = fmaxf(r.top, s_tmp[1][w]);
    return r;
}

// The 16-byte units of a head's q or k row, turned by the row's angles, in work items: an item is one unit, or with rotated halves
// of whole units the two units that turn into each other.
struct RotItems { int pairs, count; };           // pairs: of units; items of a row
template <bool ROT> LLM_DEVICE RotItems rot_items(int nu, int half) {
    const int pairs = ROT && half % 8 == 0 ? half / 8 : 0;
    return {pairs, nu - pairs};
}
// What an item of row x needs from memory; loads of several items are issued together, ahead of the arithmetic
template <bool ROT> struct RotRaw { uint4 a, b; float4 cs[4]; };
template <> struct RotRaw<false> { uint4 a; };
template <bool ROT> LLM_DEVICE void rot_load(const __nv_bfloat16* x, int i, const RotItems& it, int dim, const float2* ang, int half, RotRaw<ROT>& r) {
    if constexpr (ROT) {
        if (i < it.pairs) {
            r.a = *reinterpret_cast<const uint4*>(x + i * 8);
            r.b = *reinterpret_cast<const uint4*>(x + half + i * 8);
#pragma unroll
            for (int j = 0; j < 4; ++j) r.cs[j] = *reinterpret_cast<const float4*>(ang + i * 8 + 2 * j);     // two pairs; rows of 8 float2: 16-byte aligned
            return;
        }
        if (it.pairs == 0) return;                                   // single values: read where they are turned
    }
    const int u = i + it.pairs;
    r.a = u * 8 < dim ? *reinterpret_cast<const uint4*>(x + u * 8) : make_uint4(0, 0, 0, 0);
}
// its values (zeros behind dim): f(unit, values)
template <bool ROT, class F> LLM_DEVICE void rot_apply(const __nv_bfloat16* x, int i, const RotItems& it, int dim, const float2* ang, int half, const RotRaw<ROT>& r, F&& f) {
    auto unpack = [](const uint4& w, float (&v)[8]) {
        const uint32_t a[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) { v[2 * j] = bf16_lo(a[j]); v[2 * j + 1] = bf16_hi(a[j]); }
    };
    const int u = i + it.pairs;
    float v[8] = {};
    if constexpr (ROT) {
        if (i < it.pairs) {
            float x0[8], x1[8], y[8];
            unpack(r.a, x0);
            unpack(r.b, x1);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                v[2 * j] = x0[2 * j] * r.cs[j].x - x1[2 * j] * r.cs[j].y;
                y[2 * j] = x1[2 * j] * r.cs[j].x + x0[2 * j] * r.cs[j].y;
                v[2 * j + 1] = x0[2 * j + 1] * r.cs[j].z - x1[2 * j + 1] * r.cs[j].w;
                y[2 * j + 1] = x1[2 * j + 1] * r.cs[j].z + x0[2 * j + 1] * r.cs[j].w;
            }
            f(i, v);
            f(u, y);
            return;
        }
        if (it.pairs == 0) {
            if (u * 8 < dim) {
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] = rotated(x, u * 8 + j, ang, half);
            }
            f(u, v);
            return;
        }
    }
    unpack(r.a, v);
    f(u, v);
}
LLM_DEVICE void tmem_st8(uint32_t taddr, const uint32_t* r) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]) : "memory");
}
// two bf16 numbers whose sum is x to 16 bits of mantissa
LLM_DEVICE void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x, y);
    lo = pack_bf16(x - bf16_lo(hi), y - bf16_hi(hi));
}

LLM_DEVICE void begin_cta(uint64_t* s_bars, int n_bars, uint32_t* s_tmem, int* s_abort, int cols) {
    if (threadIdx.x == 0) {
        s_abort[0] = 0; s_abort[1] = 0;
        for (int i = 0; i < n_bars; ++i) mbar_init(smem_u32(s_bars) + i * 8, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        fence_proxy_async();
    }
    if (threadIdx.x < 32) {
        __syncwarp();
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(s_tmem)), "r"(cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
}
LLM_DEVICE void end_cta(volatile int* s_abort, int* status, uint32_t tmem, int cols) {
    tc_fence_before();
    __syncthreads();
    teardown(s_abort, threadIdx.x, status);
    if (threadIdx.x < 32) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(cols) : "memory");
}

// ---- states of single chunks ---------------------------------------------------------------------------------------------------
// D[v, d] = sum_j V[j, v] (w_j k_j)[d]: both operands are read as they lie (MN-major), rows j along K.
template <bool ROT>
__global__ void __launch_bounds__(THREADS, 2) chunk_state_kernel(const __grid_constant__ CUtensorMap map_v, const LinearParams p, const LinearChunks c) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t s_bars[2];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort[2];
    __shared__ float s_tmp[2][4], s_w[C];
    __shared__ float s_red[THREADS * 8];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int4 ck = c.chunks[blockIdx.x];
    const int h = blockIdx.y, v0 = blockIdx.z * VS, r0 = ck.x, len = ck.y;
    const int na = (p.dim + 63) / 64, nu = (p.dim + 15) / 16 * 2, n16 = nu * 8;          // operand atoms, 16-byte units and values of a k row
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t sV = base, sH = sV + 2 * ATOM, sL = sH + na * ATOM;
    const uint32_t bar_v = smem_u32(s_bars), bar_d = bar_v + 8;
    begin_cta(s_bars, 2, &s_tmem, s_abort, 128);
    const uint32_t tmem = s_tmem;
    volatile int* abort_flag = s_abort;
    pdl_wait();
    if (tid == 0) {
        mbar_arrive_expect_tx(bar_v, 2 * ATOM);
        for (int a = 0; a < 2; ++a) tma_load_3d(sV + a * ATOM, &map_v, v0 + a * 64, h, r0, bar_v);
    }
    const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(p.in) + (size_t)r0 * p.in_row + p.k_off + h * p.dim;
    const float2* ang = ROT ? p.angles + (size_t)r0 * p.half : nullptr;
    const RotItems items = rot_items<ROT>(nu, p.half);
    const int groups = THREADS / items.count, item = tid % items.count, grp = tid / items.count;
    constexpr int BATCH = ROT ? 2 : 4;
    RotRaw<ROT> raw[BATCH];
    auto load = [&](int j0) {
#pragma unroll
        for (int i = 0; i < BATCH; ++i) {
            const int j = min(j0 + i * groups, len - 1);               // rows past the chunk: any valid one, their weight is zero
            rot_load<ROT>(kp + (size_t)j * p.in_row, item, items, p.dim, ROT ? ang + (size_t)j * p.half : nullptr, p.half, raw[i]);
        }
    };
    load(grp);
    {
        const Gates g = chunk_gates(p, h, r0, len, s_tmp);
        if (p.gates && v0 == 0 && tid < C) c.gate[((size_t)blockIdx.x * p.heads + h) * C + tid] = make_float4(g.a, g.g, g.top, 0.f);
        if (tid < C) s_w[tid] = g.top;
        __syncthreads();
        const float top = s_w[len - 1];                               // A_L
        __syncthreads();
        if (tid < C) s_w[tid] = tid < len ? ex2(g.a - top) * p.k_scale : 0.f;
        if (tid == len - 1 && v0 == 0) *reinterpret_cast<float4*>(c.scal + ((size_t)blockIdx.x * p.heads + h) * 4) = make_float4(g.g, top, 0.f, 0.f);
        __syncthreads();
    }
    float sum[2][8] = {};                                             // of this thread's rows, by unit of the item
    for (int j0 = grp; j0 < C && grp < groups; j0 += BATCH * groups) {
        if (j0 != grp) load(j0);
#pragma unroll
        for (int i = 0; i < BATCH; ++i) {
            const int j = j0 + i * groups;
            if (j >= C) break;
            const float w = s_w[j];
            int part = 0;
            auto put = [&](int u, float (&v)[8]) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 8; ++e) { v[e] *= w; sum[part][e] += v[e]; }
#pragma unroll
                for (int e = 0; e < 4; ++e) split_bf16(v[2 * e], v[2 * e + 1], hi[e], lo[e]);
                st_shared_v4(atom_addr(sH + (u >> 3) * ATOM, j, u & 7), make_uint4(hi[0], hi[1], hi[2], hi[3]));
                st_shared_v4(atom_addr(sL + (u >> 3) * ATOM, j, u & 7), make_uint4(lo[0], lo[1], lo[2], lo[3]));
                part = 1;
            };
            const int r = min(j, len - 1);
            rot_apply<ROT>(kp + (size_t)r * p.in_row, item, items, p.dim, ROT ? ang + (size_t)r * p.half : nullptr, p.half, raw[i], put);
        }
    }
    if (p.gates && v0 == 0 && grp < groups) {
        if (item < items.pairs) {
#pragma unroll
            for (int e = 0; e < 8; ++e) s_red[grp * n16 + (item + items.pairs) * 8 + e] = sum[1][e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) s_red[grp * n16 + (item < items.pairs ? item : item + items.pairs) * 8 + e] = sum[0][e];
    }
    fence_proxy_async();
    __syncthreads();
    bool ok = true;
    if (warp == 0) {
        ok = mbar_wait_warp(bar_v, 0, abort_flag);
        if (ok && elect_one()) {
            const uint32_t idesc = instr_desc(n16) | (1u << 15) | (1u << 16);
            const uint64_t a = smem_desc_mn_sw128(sV, ATOM), b = smem_desc_mn_sw128(sH, ATOM), bl = smem_desc_mn_sw128(sL, ATOM);
#pragma unroll
            for (int ks = 0; ks < C / 16; ++ks) {
                mma_f16(tmem, a + ks * (2048 / 16), b + ks * (2048 / 16), idesc, ks > 0 ? 1u : 0u);
                mma_f16(tmem, a + ks * (2048 / 16), bl + ks * (2048 / 16), idesc, 1u);
            }
            mma_commit(bar_d);
        }
        __syncwarp();
    }
    if (p.gates && v0 == 0)
        for (int d = tid; d < p.dim; d += THREADS) {
            float s = 0.f;
            for (int g = 0; g < groups; ++g) s += s_red[g * n16 + d];
            c.vec[((size_t)blockIdx.x * p.heads + h) * p.dim + d] = s;
        }
    ok = ok && mbar_wait_warp(bar_d, 0, abort_flag);
    if (ok) {
        tc_fence_after();
        // through shared memory (the operands are done with): rows of 512 bytes, 16-byte units swizzled, then whole rows to memory
        const int row = (warp & 3) * 32 + lane;
        auto unit_at = [&](int r, int u) { return sV + r * 512 + (((u & ~7) | ((u ^ r) & 7)) << 4); };
        for (int c0 = (warp >> 2) * 16; c0 < n16; c0 += 32) {
            uint32_t r[16];
            tmem_ld_n<16>(tmem + ((uint32_t)((warp & 3) * 32) << 16) + c0, r);
#pragma unroll
            for (int e = 0; e < 4; ++e) st_shared_v4(unit_at(row, c0 / 4 + e), make_uint4(r[4 * e], r[4 * e + 1], r[4 * e + 2], r[4 * e + 3]));
        }
    }
    __syncthreads();
    if (ok) {
        float* dst = c.state + (((size_t)blockIdx.x * p.heads + h) * p.vdim + v0) * p.dim;
        const int rows = min(VS, p.vdim - v0);
        for (int r = warp; r < rows; r += THREADS / 32)
            if (lane * 4 < p.dim) {
                uint4 w;
                asm volatile("ld.shared.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(w.x), "=r"(w.y), "=r"(w.z), "=r"(w.w) : "r"(sV + r * 512 + (((lane & ~7) | ((lane ^ r) & 7)) << 4)));
                *reinterpret_cast<uint4*>(dst + (size_t)r * p.dim + lane * 4) = w;
            }
    }
    end_cta(s_abort, c.status, tmem, 128);
}

// ---- states in front of the chunks ---------------------------------------------------------------------------------------------
// A warp per row of the state (lanes hold four values each; the row past the last is the normaliser n).  The chunk's own sum is
// replaced by the state in front of it, as [hi | lo] bf16 halves of the row.
constexpr int SCAN_WARPS = 8, AHEAD = 4;
__global__ void __launch_bounds__(32 * SCAN_WARPS) chunk_scan_kernel(const LinearParams p, const LinearChunks c) {
    pdl_wait();
    const int lane = threadIdx.x & 31, row = blockIdx.x * SCAN_WARPS + (threadIdx.x >> 5), h = blockIdx.y;
    const bool lstm = p.gates != nullptr, is_n = row == p.vdim;
    if (row > p.vdim || (is_n && !lstm)) return;
    const int4 sq = c.seqs[blockIdx.z];
    const int slot = LLM_CHECK_INDEX(p.slots[blockIdx.z], p.n_slots), c0 = sq.x, n = sq.y, d = lane * 4;
    const bool fresh = p.positions[c.chunks[c0].x] == 0, live = d < p.dim;
    float* pool = is_n ? p.n + ((size_t)slot * p.heads + h) * p.dim : p.S + (((size_t)slot * p.heads + h) * p.vdim + row) * p.dim;
    float* m_pool = lstm ? p.m + (size_t)slot * p.heads + h : nullptr;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!fresh && live) s = *reinterpret_cast<const float4*>(pool + d);
    float m = lstm && !fresh ? *m_pool * LOG2E : 0.f;
    __syncwarp();
    auto at = [&](int i) { return is_n ? c.vec + ((size_t)(c0 + i) * p.heads + h) * p.dim : c.state + (((size_t)(c0 + i) * p.heads + h) * p.vdim + row) * p.dim; };
    auto scal = [&](int i) { return c.scal + ((size_t)(c0 + i) * p.heads + h) * 4; };
    float4 kv[AHEAD];
    float2 sc[AHEAD];
    auto fetch = [&](int i, float4& x, float2& y) {
        if (i >= n) return;
        if (live) x = __ldcg(reinterpret_cast<const float4*>(at(i) + d));
        y = __ldcg(reinterpret_cast<const float2*>(scal(i)));
    };
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) { kv[i] = s; fetch(i, kv[i], sc[i]); }
    for (int i0 = 0; i0 < n; i0 += AHEAD) {
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (i0 + i >= n) break;
            const float4 x = kv[i];
            const float2 y = sc[i];
            fetch(i0 + i + AHEAD, kv[i], sc[i]);
            float keep, add = 1.f;
            if (lstm) {
                const float top = fmaxf(m, y.y);
                if (is_n && lane == 0) scal(i0 + i)[2] = m;               // stabiliser of the state in front of the chunk
                keep = ex2(m - top);
                add = ex2(y.y - top);
                m = y.x + top;
            } else {
                keep = ex2(y.x);
            }
            const float4 next = make_float4(keep * s.x + add * x.x, keep * s.y + add * x.y, keep * s.z + add * x.z, keep * s.w + add * x.w);
            __syncwarp();                                            // the whole row has been read
            if (live) {
                if (is_n) {
                    *reinterpret_cast<float4*>(at(i0 + i) + d) = s;
                } else {
                    uint32_t h0, l0, h1, l1;
                    split_bf16(s.x, s.y, h0, l0);
                    split_bf16(s.z, s.w, h1, l1);
                    __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(at(i0 + i));
                    *reinterpret_cast<uint2*>(dst + d) = make_uint2(h0, h1);
                    *reinterpret_cast<uint2*>(dst + p.dim + d) = make_uint2(l0, l1);
                }
            }
            s = next;
        }
    }
    if (live) *reinterpret_cast<float4*>(pool + d) = s;
}
// (chunk_out runs behind chunk_scan and in front of any other use of the slots: the new stabilisers can be stored by it)

// ---- outputs --------------------------------------------------------------------------------------------------------------------
// A CTA takes 256 values of a head (all of most heads) in two slices, so that the weights are computed once.  Shared memory, in atoms:
// Q [na] | K, then V of slice 1 [2] | V of slice 0, then gate of slice 1 [2] | state [2 na: hi, lo], of one slice after the other |
// gate of slice 0 [2].  With the whole head here (`fused`) the norm and the gate follow, otherwise head_gate does them (`raw`: nobody).
constexpr int T_S = 0, T_P = 128, T_O = 256, T_I = 384;              // TMEM columns: scores (then T_I of slice 1), weights (hi, lo), both parts of o
// (a barrier that is waited for twice is not used again before every thread has seen its first phase)
enum OBar { B_QK = 0, B_V, B_V1, B_G, B_G1, B_ST, B_SC, B_IN, B_IN1, B_O, N_OBARS };

template <bool ROT>
__global__ void __launch_bounds__(THREADS, 1) chunk_out_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                                               const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_g,
                                                               const __grid_constant__ CUtensorMap map_s, const LinearParams p, const LinearChunks c) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t s_bars[N_OBARS];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort[2];
    __shared__ float s_top[C], s_keep[C], s_floor[C], s_x[2][C], s_y[2][C];
    __shared__ __align__(16) float s_a[C], s_n[128];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int4 ck = c.chunks[blockIdx.x];
    const int h = blockIdx.y, v0 = blockIdx.z * 2 * VS, r0 = ck.x, len = ck.y;
    const int na = (p.dim + 63) / 64, nkv = max(na, 2), ksteps = (p.dim + 15) / 16;
    const int slices = p.vdim - v0 > VS ? 2 : 1;
    const bool lstm = p.gates != nullptr, fused = gridDim.z == 1 && !p.raw;
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t sQ = base, sK = sQ + na * ATOM, sV = sK + nkv * ATOM, sS = sV + 2 * ATOM, sG = sS + 2 * na * ATOM;
    const uint32_t bars = smem_u32(s_bars);
    auto bar = [&](int i) { return bars + i * 8; };
    auto width = [&](int s) { return min(VS, (p.vdim - v0 - s * VS + 15) / 16 * 16); };       // values of slice s, whole MMA steps
    auto load_rows = [&](uint32_t dst, const CUtensorMap* map, int s, int b) {                 // [rows][128 values of slice s]
        mbar_arrive_expect_tx(bar(b), 2 * ATOM);
        for (int a = 0; a < 2; ++a) tma_load_3d(dst + a * ATOM, map, v0 + s * VS + a * 64, h, r0, bar(b));
    };
    auto load_state = [&](int s) {
        mbar_arrive_expect_tx(bar(B_ST), 2 * na * ATOM);
        for (int part = 0; part < 2; ++part)
            for (int a = 0; a < na; ++a) tma_load_4d(sS + (part * na + a) * ATOM, &map_s, a * 64, part, v0 + s * VS, blockIdx.x * p.heads + h, bar(B_ST));
    };
    begin_cta(s_bars, N_OBARS, &s_tmem, s_abort, 512);
    const uint32_t tmem = s_tmem;
    volatile int* abort_flag = s_abort;
    pdl_wait();
    if (tid == 0) {
        if (!ROT) {
            mbar_arrive_expect_tx(bar(B_QK), 2 * na * ATOM);
            for (int a = 0; a < na; ++a) {
                tma_load_3d(sQ + a * ATOM, &map_q, a * 64, h, r0, bar(B_QK));
                tma_load_3d(sK + a * ATOM, &map_k, a * 64, h, r0, bar(B_QK));
            }
        }
        load_state(0);
        load_rows(sV, &map_v, 0, B_V);
        if (fused) load_rows(sG, &map_g, 0, B_G);
    }
    if constexpr (ROT) {
        const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(p.in) + (size_t)r0 * p.in_row + h * p.dim;
        const RotItems items = rot_items<true>(ksteps * 2, p.half);
        const int n = 2 * items.count, groups = THREADS / n, which = tid % n >= items.count, item = tid % n - which * items.count;
        const uint32_t dst = which ? sK : sQ;
        const __nv_bfloat16* x = in + (which ? p.k_off : p.q_off);
        constexpr int BATCH = 4;
        for (int j0 = tid / n; j0 < C && tid / n < groups; j0 += BATCH * groups) {
            RotRaw<true> raw[BATCH];
            // rows past the chunk repeat its last one (their results are not stored)
            auto at = [&](int i) { return min(j0 + i * groups, len - 1); };
#pragma unroll
            for (int i = 0; i < BATCH; ++i) rot_load<true>(x + (size_t)at(i) * p.in_row, item, items, p.dim, p.angles + (size_t)(r0 + at(i)) * p.half, p.half, raw[i]);
#pragma unroll
            for (int i = 0; i < BATCH; ++i) {
                const int j = j0 + i * groups;
                if (j >= C) break;
                auto put = [&](int u, float (&v)[8]) {
                    st_shared_v4(atom_addr(dst + (u >> 3) * ATOM, j, u & 7),
                                 make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7])));
                };
                rot_apply<true>(x + (size_t)at(i) * p.in_row, item, items, p.dim, p.angles + (size_t)(r0 + at(i)) * p.half, p.half, raw[i], put);
            }
        }
    }
    {
        if (tid < C) {
            Gates g = {-INFINITY, 0.f, -INFINITY};
            if (lstm) {
                const float4 x = __ldcg(c.gate + ((size_t)blockIdx.x * p.heads + h) * C + tid);
                g = {x.x, x.y, x.z};
            } else if (tid < len) {
                g = retention_gates(p.decay[h], tid);
            }
            const float m = lstm ? __ldcg(c.scal + ((size_t)blockIdx.x * p.heads + h) * 4 + 2) : 0.f;
            const float top = lstm ? fmaxf(m, g.top) : g.top;
            s_a[tid] = g.a;
            s_top[tid] = tid < len ? top : 0.f;
            s_keep[tid] = tid < len ? (lstm ? ex2(m - top) : ex2(g.g)) * p.q_scale : 0.f;
            s_floor[tid] = ex2(-(g.g + top));
        }
        if (lstm) for (int d = tid; d < p.dim; d += THREADS) s_n[d] = __ldcg(c.vec + ((size_t)blockIdx.x * p.heads + h) * p.dim + d);
    }
    if (ROT) fence_proxy_async();
    __syncthreads();
    bool ok = true;
    // one warp issues: o's part from the state of slice s into column t_i
    auto issue_in = [&](int s, uint32_t t_i) {
        ok = ok && mbar_wait_warp(bar(B_ST), s, abort_flag);
        if (ok && elect_one()) {
            const uint64_t q = smem_desc_sw128(sQ), st = smem_desc_sw128(sS);
            const uint32_t idesc = instr_desc(width(s));
            for (int ks = 0; ks < ksteps; ++ks) {
                const uint32_t off = (ks >> 2) * (ATOM / 16) + 2 * (ks & 3);
                mma_f16(tmem + t_i, q + off, st + off, idesc, ks > 0 ? 1u : 0u);
                mma_f16(tmem + t_i, q + off, st + off + na * (ATOM / 16), idesc, 1u);
            }
            mma_commit(bar(s ? B_IN1 : B_IN));
        }
        __syncwarp();
    };
    auto issue_o = [&](int s) {
        ok = ok && mbar_wait_warp(bar(s ? B_V1 : B_V), 0, abort_flag);
        tc_fence_after();
        if (ok && elect_one()) {
            const uint64_t v = smem_desc_mn_sw128(s ? sK : sV, ATOM);
            const uint32_t idesc = instr_desc(width(s)) | (1u << 16);
#pragma unroll
            for (int ks = 0; ks < C / 16; ++ks) {
                mma_f16_ts(tmem + T_O, tmem + T_P + ks * 8, v + ks * (2048 / 16), idesc, ks > 0 ? 1u : 0u);
                mma_f16_ts(tmem + T_O, tmem + T_P + 64 + ks * 8, v + ks * (2048 / 16), idesc, 1u);
            }
            mma_commit(bar(B_O));
        }
        __syncwarp();
    };
    if (warp == 0) {
        if (!ROT) ok = mbar_wait_warp(bar(B_QK), 0, abort_flag);
        if (ok && elect_one()) {
            const uint64_t q = smem_desc_sw128(sQ), k = smem_desc_sw128(sK);
            for (int ks = 0; ks < ksteps; ++ks) {
                const uint32_t off = (ks >> 2) * (ATOM / 16) + 2 * (ks & 3);
                mma_f16(tmem + T_S, q + off, k + off, instr_desc(C), ks > 0 ? 1u : 0u);
            }
            mma_commit(bar(B_SC));
        }
        __syncwarp();
        issue_in(0, T_I);
    }
    // weights: two threads per row (= TMEM lane), 64 columns each
    const int row = (warp & 3) * 32 + lane, half = warp >> 2;
    const uint32_t t_lane = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    if (!ROT) ok = ok && mbar_wait_warp(bar(B_QK), 0, abort_flag);       // the dot products with n read the queries
    ok = ok && mbar_wait_warp(bar(B_SC), 0, abort_flag);
    if (ok) {
        tc_fence_after();
        if (slices == 2 && tid == 0) load_rows(sK, &map_v, 1, B_V1);      // the keys are done with
        __syncwarp();
        const float top = s_top[row], scale = p.q_scale * p.k_scale;
        float sum = 0.f;
        const bool none = half * 64 > (warp & 3) * 32 + 31;              // nothing here for this warp's rows
        // (rolled loops here and below: every instruction of a CTA is fetched once, and straight-line code of this size waited for that)
#pragma unroll 1
        for (int q = 0; q < 4; ++q) {
            uint32_t r[16], hl[16];                                      // hl: hi words, then lo words
            if (!none) {
                tmem_ld_n<16>(t_lane + T_S + half * 64 + q * 16, r);
#pragma unroll
                for (int i = 0; i < 16; i += 4) {
                    const int j = half * 64 + q * 16 + i;
                    const float4 a = *reinterpret_cast<const float4*>(s_a + j);
                    const float e[4] = {a.x, a.y, a.z, a.w};
                    float w[4];
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        w[x] = j + x <= row ? __uint_as_float(r[i + x]) * scale * ex2(e[x] - top) : 0.f;
                        sum += w[x];
                    }
                    split_bf16(w[0], w[1], hl[i / 2], hl[8 + i / 2]);
                    split_bf16(w[2], w[3], hl[i / 2 + 1], hl[8 + i / 2 + 1]);
                }
            } else {
#pragma unroll
                for (int i = 0; i < 16; ++i) hl[i] = 0u;
            }
            tmem_st8(t_lane + T_P + half * 32 + q * 8, hl);
            tmem_st8(t_lane + T_P + 64 + half * 32 + q * 8, hl + 8);
        }
        if (lstm) {
            float dot = 0.f;
            for (int u = half; u * 8 < p.dim; u += 2) {
                uint4 w;
                asm volatile("ld.shared.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(w.x), "=r"(w.y), "=r"(w.z), "=r"(w.w) : "r"(atom_addr(sQ + (u >> 3) * ATOM, row, u & 7)));
                const uint32_t x[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) dot += bf16_lo(x[e]) * s_n[u * 8 + 2 * e] + bf16_hi(x[e]) * s_n[u * 8 + 2 * e + 1];
            }
            sum += dot * s_keep[row];
        }
        s_x[half][row] = sum;
        tmem_wait_st();
        tc_fence_before();
    }
    __syncthreads();                                                     // weights are in place, the scores have been read
    if (warp == 0) {
        issue_o(0);
        if (slices == 2) {
            ok = ok && mbar_wait_warp(bar(B_IN), 0, abort_flag);         // the state of slice 0 is done with
            if (ok && elect_one()) load_state(1);
            __syncwarp();
        }
    }
    const float keep = s_keep[row];
    const float inv = lstm ? 1.f / (fmaxf(fabsf(s_x[0][row] + s_x[1][row]), s_floor[row]) + NORM_FLOOR) : 1.f;
    float ss = 0.f;
    // both parts of o together; the sums stay in tensor memory (columns T_I of slice 0, T_O of slice 1) until the norm is known
#pragma unroll 1
    for (int s = 0; s < slices; ++s) {
        ok = ok && mbar_wait_warp(bar(s ? B_IN1 : B_IN), 0, abort_flag) && mbar_wait_warp(bar(B_O), s, abort_flag);
        if (ok) {
            tc_fence_after();
            if (fused && s == 0 && slices == 2 && tid == 0) load_rows(sV, &map_g, 1, B_G1);       // the values of slice 0 are done with
            __syncwarp();
            const int w = width(s);
#pragma unroll 1
            for (int c0 = half * 64; c0 < min(w, half * 64 + 64); c0 += 16) {        // the same for all threads of the warp
                uint32_t a[16], b[16];
                tmem_ld_n<16>(t_lane + T_O + c0, a);
                tmem_ld_n<16>(t_lane + (s ? T_S : T_I) + c0, b);
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float x = (__uint_as_float(a[i]) + keep * __uint_as_float(b[i])) * inv;
                    ss += x * x;
                    a[i] = __float_as_uint(x);
                }
                tmem_st_n<16>(t_lane + (s ? T_O : T_I) + c0, a);
            }
            tmem_wait_st();
            tc_fence_before();
        }
        if (s == 0 && slices == 2) {
            __syncthreads();                                             // slice 0 has been read out of T_O
            if (warp == 0) {
                issue_in(1, T_S);
                issue_o(1);
            }
        }
    }
    s_y[half][row] = ss;
    __syncthreads();
    const float rms = fused ? 1.f / sqrtf((s_y[0][row] + s_y[1][row]) / (float)p.true_vdim + p.eps) : 1.f;
#pragma unroll 1
    for (int s = 0; s < slices; ++s) {
        // gated values into the gate's own place (fused), or o as it is; then whole rows to memory
        const uint32_t tile = s ? sV : sG;
        if (fused) ok = ok && mbar_wait_warp(bar(s ? B_G1 : B_G), 0, abort_flag);
        const int w = width(s);
        if (ok) {
#pragma unroll 1
            for (int c0 = half * 64; c0 < min(w, half * 64 + 64); c0 += 16) {
                uint32_t o[16];
                tmem_ld_n<16>(t_lane + (s ? T_O : T_I) + c0, o);
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    const uint32_t at = atom_addr(tile + half * ATOM, row, (c0 & 63) / 8 + k);
                    float v[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(o[k * 8 + i]);
                    if (fused) {
                        uint32_t g[4];
                        asm volatile("ld.shared.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(g[0]), "=r"(g[1]), "=r"(g[2]), "=r"(g[3]) : "r"(at));
                        const int col = v0 + s * VS + c0 + k * 8;
                        float4 n0 = make_float4(1.f, 1.f, 1.f, 1.f), n1 = n0;
                        if (p.norm_w && col < p.vdim) {
                            n0 = *reinterpret_cast<const float4*>(p.norm_w + h * p.vdim + col);
                            n1 = *reinterpret_cast<const float4*>(p.norm_w + h * p.vdim + col + 4);
                        }
                        const float n[8] = {n0.x, n0.y, n0.z, n0.w, n1.x, n1.y, n1.z, n1.w};
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            const float z = i & 1 ? bf16_hi(g[i >> 1]) : bf16_lo(g[i >> 1]);
                            v[i] *= rms * n[i] * (p.silu ? z : 1.f) * __fdividef(1.f, 1.f + __expf(-z));
                        }
                    }
                    st_shared_v4(at, make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7])));
                }
            }
        }
        __syncthreads();
        if (ok) {
            __nv_bfloat16* dst = (fused ? static_cast<__nv_bfloat16*>(p.out) + (size_t)r0 * p.out_row : c.o + (size_t)r0 * p.heads * p.vdim) + (size_t)h * p.vdim + v0 + s * VS;
            const size_t stride = fused ? p.out_row : (size_t)p.heads * p.vdim;
            const int u = lane & 15;
            for (int r = warp * 2 + (lane >> 4); r < len; r += THREADS / 16)
                if (v0 + s * VS + u * 8 < p.vdim) {
                    uint4 x;
                    asm volatile("ld.shared.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(x.x), "=r"(x.y), "=r"(x.z), "=r"(x.w) : "r"(atom_addr(tile + (u >> 3) * ATOM, r, u & 7)));
                    *reinterpret_cast<uint4*>(dst + (size_t)r * stride + u * 8) = x;
                }
        }
    }
    // the stabiliser behind the sequence's last chunk
    if (lstm && v0 == 0 && ck.w && tid == 0) {
        const float* sc = c.scal + ((size_t)blockIdx.x * p.heads + h) * 4;
        p.m[(size_t)LLM_CHECK_INDEX(p.slots[ck.z], p.n_slots) * p.heads + h] = (sc[0] + fmaxf(sc[2], sc[1])) * (1.f / LOG2E);
    }
    end_cta(s_abort, c.status, tmem, 512);
}

static size_t state_smem(int dim) { return (size_t)(2 + 2 * ((dim + 63) / 64)) * ATOM + 1024; }       // at least the 64 KB of the staged result
static size_t out_smem(int dim) {
    const int na = (dim + 63) / 64;
    return (size_t)(3 * na + (na > 2 ? na : 2) + 4) * ATOM + 1024;
}

}  // namespace lin

bool linear_chunk_fits(int dim, int vdim) { return dim % 8 == 0 && vdim % 8 == 0 && dim >= 8 && dim <= 128 && vdim >= 8; }

cudaError_t launch_linear_chunk(const LinearParams& p, const LinearChunks& c, cudaStream_t st) {
    using namespace lin;
    if (c.n_chunks == 0) return cudaSuccess;
    if (!linear_chunk_fits(p.dim, p.vdim) || p.in_row % 8 || p.q_off % 8 || p.k_off % 8 || p.v_off % 8 || p.g_off % 8 || p.out_row % 8 || p.silu_in || p.heads > 65535 || c.n_seqs > 65535 ||
        (!p.gates == !p.decay) || (p.gates && p.half))
        return cudaErrorInvalidValue;
    const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(p.in);
    CUtensorMap mq, mk, mv, mg, ms;
    auto rows_map = [&](CUtensorMap* m, int off, int size) {             // [T][heads][size]
        const cuuint64_t dims[3] = {(cuuint64_t)size, (cuuint64_t)p.heads, (cuuint64_t)c.rows}, strides[2] = {(cuuint64_t)size, (cuuint64_t)p.in_row};
        const cuuint32_t box[3] = {64, 1, C};
        return make_map_nd<3>(m, in + off, dims, strides, box);
    };
    const cuuint64_t sd[4] = {(cuuint64_t)p.dim, 2, (cuuint64_t)p.vdim, (cuuint64_t)c.n_chunks * p.heads};
    const cuuint64_t ss[3] = {(cuuint64_t)p.dim, (cuuint64_t)2 * p.dim, (cuuint64_t)2 * p.dim * p.vdim};
    const cuuint32_t sb[4] = {64, 1, VS, 1};
    if (!rows_map(&mq, p.q_off, p.dim) || !rows_map(&mk, p.k_off, p.dim) || !rows_map(&mv, p.v_off, p.vdim) ||
        !rows_map(&mg, p.g_off, p.vdim) || !make_map_nd<4>(&ms, c.state, sd, ss, sb))
        return cudaErrorInvalidValue;
    const bool rot = p.half > 0;
    const dim3 grid(c.n_chunks, p.heads, (p.vdim + VS - 1) / VS), out_grid(c.n_chunks, p.heads, (p.vdim + 2 * VS - 1) / (2 * VS));
    cudaError_t e;
    auto state = [&](auto kernel) {
        e = raise_smem(kernel, state_smem(p.dim));
        return e != cudaSuccess ? e : launch_pdl(kernel, grid, dim3(THREADS), state_smem(p.dim), st, mv, p, c);
    };
    e = rot ? state(chunk_state_kernel<true>) : state(chunk_state_kernel<false>);
    if (e != cudaSuccess) return e;
    e = launch_pdl(chunk_scan_kernel, dim3(p.vdim / SCAN_WARPS + 1, p.heads, c.n_seqs), dim3(32 * SCAN_WARPS), 0, st, p, c);
    if (e != cudaSuccess) return e;
    auto out = [&](auto kernel) {
        e = raise_smem(kernel, out_smem(p.dim));
        return e != cudaSuccess ? e : launch_pdl(kernel, out_grid, dim3(THREADS), out_smem(p.dim), st, mq, mk, mv, mg, ms, p, c);
    };
    e = rot ? out(chunk_out_kernel<true>) : out(chunk_out_kernel<false>);
    return e != cudaSuccess || p.raw || out_grid.z == 1 ? e : launch_head_gate(p, c.o, c.rows, st);
}

int bounds_status_linear_tc(bool reset);
LLM_DEFINE_BOUNDS_STATUS_READER(bounds_status_linear_tc)

}  // namespace llm
