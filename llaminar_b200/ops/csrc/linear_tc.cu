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
//   chunk_out     per chunk and head: scores, weights, o                     tcgen05, M = 128 rows, N = 128 rows / values
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
LLM_DEVICE Gates chunk_gates(const LinearParams& p, int h, int r0, int len, float (&s_tmp)[2][4]) {
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5;
    Gates r = {-INFINITY, 0.f, -INFINITY};
    if (!p.gates) {
        const float l = log2_decay(p.decay[h]);
        if (t < len) { r.g = (float)(t + 1) * l; r.a = -r.g; r.top = r.a; }
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

// values u * 8 .. u * 8 + 7 of head vector x (dim values), turned by the row's angles
LLM_DEVICE void head_unit(const __nv_bfloat16* x, int u, int dim, const float2* ang, int half, float (&v)[8]) {
    const int i0 = u * 8;
    if (half % 8 == 0 && i0 < 2 * half) {
        const bool first = i0 < half;
        const int a0 = first ? i0 : i0 - half;
        const uint4 own = *reinterpret_cast<const uint4*>(x + i0), other = *reinterpret_cast<const uint4*>(x + (first ? i0 + half : i0 - half));
        const uint32_t a[4] = {own.x, own.y, own.z, own.w}, b[4] = {other.x, other.y, other.z, other.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 c0 = ang[a0 + 2 * j], c1 = ang[a0 + 2 * j + 1];
            v[2 * j] = bf16_lo(a[j]) * c0.x + bf16_lo(b[j]) * (first ? -c0.y : c0.y);
            v[2 * j + 1] = bf16_hi(a[j]) * c1.x + bf16_hi(b[j]) * (first ? -c1.y : c1.y);
        }
    } else if (i0 >= 2 * half) {
        const uint4 own = *reinterpret_cast<const uint4*>(x + i0);
        const uint32_t a[4] = {own.x, own.y, own.z, own.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) { v[2 * j] = bf16_lo(a[j]); v[2 * j + 1] = bf16_hi(a[j]); }
    } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = rotated(x, i0 + j, ang, half);
    }
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
    {
        const Gates g = chunk_gates(p, h, r0, len, s_tmp);
        if (tid < C) s_w[tid] = g.top;
        __syncthreads();
        const float top = s_w[len - 1];                               // A_L
        __syncthreads();
        if (tid < C) s_w[tid] = tid < len ? ex2(g.a - top) * p.k_scale : 0.f;
        if (tid == len - 1 && v0 == 0) *reinterpret_cast<float4*>(c.scal + ((size_t)blockIdx.x * p.heads + h) * 4) = make_float4(g.g, top, 0.f, 0.f);
        __syncthreads();
    }
    const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(p.in) + (size_t)r0 * p.in_row + p.k_off + h * p.dim;
    const int groups = THREADS / nu, u = tid % nu, grp = tid / nu;
    float sum[8] = {};
    for (int j = grp; j < C && grp < groups; j += groups) {
        float v[8] = {};
        if (j < len && u * 8 < p.dim) {
            head_unit(kp + (size_t)j * p.in_row, u, p.dim, ROT ? p.angles + (size_t)(r0 + j) * p.half : nullptr, ROT ? p.half : 0, v);
            const float w = s_w[j];
#pragma unroll
            for (int e = 0; e < 8; ++e) { v[e] *= w; sum[e] += v[e]; }
        }
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split_bf16(v[2 * e], v[2 * e + 1], hi[e], lo[e]);
        st_shared_v4(atom_addr(sH + (u >> 3) * ATOM, j, u & 7), make_uint4(hi[0], hi[1], hi[2], hi[3]));
        st_shared_v4(atom_addr(sL + (u >> 3) * ATOM, j, u & 7), make_uint4(lo[0], lo[1], lo[2], lo[3]));
    }
    if (p.gates && v0 == 0 && grp < groups) {
#pragma unroll
        for (int e = 0; e < 8; ++e) s_red[grp * n16 + u * 8 + e] = sum[e];
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
        const int row = v0 + (warp & 3) * 32 + lane;
        float* dst = c.state + (((size_t)blockIdx.x * p.heads + h) * p.vdim + row) * p.dim;
        for (int c0 = (warp >> 2) * 16; c0 < n16; c0 += 32) {
            uint32_t r[16];
            tmem_ld_n<16>(tmem + ((uint32_t)((warp & 3) * 32) << 16) + c0, r);
            if (row < p.vdim)
#pragma unroll
                for (int e = 0; e < 16; e += 4)
                    if (c0 + e < p.dim) *reinterpret_cast<uint4*>(dst + c0 + e) = make_uint4(r[e], r[e + 1], r[e + 2], r[e + 3]);
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
constexpr int T_S = 0, T_P = 128, T_O = 256, T_I = 384;              // TMEM columns: scores, weights (hi, lo), both parts of o
enum OBar { B_QK = 0, B_V, B_ST, B_SC, B_IN, B_O, N_OBARS };

template <bool ROT>
__global__ void __launch_bounds__(THREADS, 1) chunk_out_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                                               const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_s,
                                                               const LinearParams p, const LinearChunks c) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t s_bars[N_OBARS];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort[2];
    __shared__ float s_tmp[2][4], s_top[C], s_keep[C], s_floor[C], s_x[2][C];
    __shared__ __align__(16) float s_a[C], s_n[128];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int4 ck = c.chunks[blockIdx.x];
    const int h = blockIdx.y, v0 = blockIdx.z * VS, r0 = ck.x, len = ck.y;
    const int na = (p.dim + 63) / 64, ksteps = (p.dim + 15) / 16, nv = min(VS, (p.vdim - v0 + 15) / 16 * 16);
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t sQ = base, sK = sQ + na * ATOM, sV = sK + na * ATOM, sS = sV + 2 * ATOM;      // sS: hi atoms, then lo
    const uint32_t bars = smem_u32(s_bars);
    auto bar = [&](int i) { return bars + i * 8; };
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
        mbar_arrive_expect_tx(bar(B_ST), 2 * na * ATOM);
        for (int part = 0; part < 2; ++part)
            for (int a = 0; a < na; ++a) tma_load_4d(sS + (part * na + a) * ATOM, &map_s, a * 64, part, v0, blockIdx.x * p.heads + h, bar(B_ST));
        mbar_arrive_expect_tx(bar(B_V), 2 * ATOM);
        for (int a = 0; a < 2; ++a) tma_load_3d(sV + a * ATOM, &map_v, v0 + a * 64, h, r0, bar(B_V));
    }
    if constexpr (ROT) {
        const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(p.in) + (size_t)r0 * p.in_row + h * p.dim;
        const int nu = ksteps * 2;
        for (int i = tid; i < 2 * C * nu; i += THREADS) {
            const int which = i / (C * nu), x = i - which * C * nu, j = x / nu, u = x - j * nu;
            float v[8] = {};
            if (j < len && u * 8 < p.dim) head_unit(in + (size_t)j * p.in_row + (which ? p.k_off : p.q_off), u, p.dim, p.angles + (size_t)(r0 + j) * p.half, p.half, v);
            st_shared_v4(atom_addr((which ? sK : sQ) + (u >> 3) * ATOM, j, u & 7),
                         make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7])));
        }
    }
    const bool lstm = p.gates != nullptr;
    {
        const Gates g = chunk_gates(p, h, r0, len, s_tmp);
        if (tid < C) {
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
    if (warp == 0) {
        if (!ROT) ok = mbar_wait_warp(bar(B_QK), 0, abort_flag);
        const uint64_t q = smem_desc_sw128(sQ), k = smem_desc_sw128(sK), s = smem_desc_sw128(sS);
        if (ok && elect_one()) {
            for (int ks = 0; ks < ksteps; ++ks) {
                const uint32_t off = (ks >> 2) * (ATOM / 16) + 2 * (ks & 3);
                mma_f16(tmem + T_S, q + off, k + off, instr_desc(C), ks > 0 ? 1u : 0u);
            }
            mma_commit(bar(B_SC));
        }
        __syncwarp();
        ok = ok && mbar_wait_warp(bar(B_ST), 0, abort_flag);
        if (ok && elect_one()) {
            for (int ks = 0; ks < ksteps; ++ks) {
                const uint32_t off = (ks >> 2) * (ATOM / 16) + 2 * (ks & 3);
                mma_f16(tmem + T_I, q + off, s + off, instr_desc(nv), ks > 0 ? 1u : 0u);
                mma_f16(tmem + T_I, q + off, s + off + na * (ATOM / 16), instr_desc(nv), 1u);
            }
            mma_commit(bar(B_IN));
        }
        __syncwarp();
    }
    // weights: two threads per row (= TMEM lane), 64 columns each
    const int row = (warp & 3) * 32 + lane, half = warp >> 2;
    const uint32_t t_lane = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    if (!ROT) ok = ok && mbar_wait_warp(bar(B_QK), 0, abort_flag);       // the dot products with n read the queries
    ok = ok && mbar_wait_warp(bar(B_SC), 0, abort_flag);
    if (ok) {
        tc_fence_after();
        const float top = s_top[row], scale = p.q_scale * p.k_scale;
        float sum = 0.f;
        uint32_t hi[32], lo[32];
        if (half * 64 > (warp & 3) * 32 + 31) {                          // nothing here for this warp's rows
#pragma unroll
            for (int i = 0; i < 32; ++i) hi[i] = lo[i] = 0u;
        } else {
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                uint32_t r[32];
                tmem_ld_n<32>(t_lane + T_S + half * 64 + q * 32, r);
#pragma unroll
                for (int i = 0; i < 32; i += 4) {
                    const int j = half * 64 + q * 32 + i;
                    const float4 a = *reinterpret_cast<const float4*>(s_a + j);
                    const float e[4] = {a.x, a.y, a.z, a.w};
                    float w[4];
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        w[x] = j + x <= row ? __uint_as_float(r[i + x]) * scale * ex2(e[x] - top) : 0.f;
                        sum += w[x];
                    }
                    split_bf16(w[0], w[1], hi[q * 16 + i / 2], lo[q * 16 + i / 2]);
                    split_bf16(w[2], w[3], hi[q * 16 + i / 2 + 1], lo[q * 16 + i / 2 + 1]);
                }
            }
        }
        tmem_st32(t_lane + T_P + half * 32, hi);
        tmem_st32(t_lane + T_P + 64 + half * 32, lo);
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
    __syncthreads();
    if (warp == 0) {
        ok = ok && mbar_wait_warp(bar(B_V), 0, abort_flag);
        tc_fence_after();
        if (ok && elect_one()) {
            const uint64_t v = smem_desc_mn_sw128(sV, ATOM);
            const uint32_t idesc = instr_desc(nv) | (1u << 16);
#pragma unroll
            for (int ks = 0; ks < C / 16; ++ks) {
                mma_f16_ts(tmem + T_O, tmem + T_P + ks * 8, v + ks * (2048 / 16), idesc, ks > 0 ? 1u : 0u);
                mma_f16_ts(tmem + T_O, tmem + T_P + 64 + ks * 8, v + ks * (2048 / 16), idesc, 1u);
            }
            mma_commit(bar(B_O));
        }
        __syncwarp();
    }
    ok = ok && mbar_wait_warp(bar(B_IN), 0, abort_flag) && mbar_wait_warp(bar(B_O), 0, abort_flag);
    if (ok) {
        tc_fence_after();
        const float keep = s_keep[row];
        const float inv = lstm ? 1.f / (fmaxf(fabsf(s_x[0][row] + s_x[1][row]), s_floor[row]) + NORM_FLOOR) : 1.f;
        __nv_bfloat16* dst = c.o + (size_t)(r0 + row) * p.heads * p.vdim + (size_t)h * p.vdim + v0;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const int c0 = half * 64 + q * 16;
            if (c0 >= nv) break;                                         // the same for all threads of the warp
            uint32_t a[16], b[16];
            tmem_ld_n<16>(t_lane + T_O + c0, a);
            tmem_ld_n<16>(t_lane + T_I + c0, b);
            uint32_t w[8];
#pragma unroll
            for (int i = 0; i < 8; ++i)
                w[i] = pack_bf16((__uint_as_float(a[2 * i]) + keep * __uint_as_float(b[2 * i])) * inv, (__uint_as_float(a[2 * i + 1]) + keep * __uint_as_float(b[2 * i + 1])) * inv);
            if (row < len) {
                if (v0 + c0 < p.vdim) *reinterpret_cast<uint4*>(dst + c0) = make_uint4(w[0], w[1], w[2], w[3]);
                if (v0 + c0 + 8 < p.vdim) *reinterpret_cast<uint4*>(dst + c0 + 8) = make_uint4(w[4], w[5], w[6], w[7]);
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

static size_t state_smem(int dim) { return (size_t)(2 + 2 * ((dim + 63) / 64)) * ATOM + 1024; }
static size_t out_smem(int dim) { return (size_t)(2 + 4 * ((dim + 63) / 64)) * ATOM + 1024; }

}  // namespace lin

bool linear_chunk_fits(int dim, int vdim) { return dim % 8 == 0 && vdim % 8 == 0 && dim >= 8 && dim <= 128 && vdim >= 8; }

cudaError_t launch_linear_chunk(const LinearParams& p, const LinearChunks& c, cudaStream_t st) {
    using namespace lin;
    if (c.n_chunks == 0) return cudaSuccess;
    if (!linear_chunk_fits(p.dim, p.vdim) || p.in_row % 8 || p.q_off % 8 || p.k_off % 8 || p.v_off % 8 || p.heads > 65535 || c.n_seqs > 65535 ||
        (!p.gates == !p.decay))
        return cudaErrorInvalidValue;
    const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(p.in);
    CUtensorMap mq, mk, mv, ms;
    auto rows_map = [&](CUtensorMap* m, int off, int size) {             // [T][heads][size]
        const cuuint64_t dims[3] = {(cuuint64_t)size, (cuuint64_t)p.heads, (cuuint64_t)c.rows}, strides[2] = {(cuuint64_t)size, (cuuint64_t)p.in_row};
        const cuuint32_t box[3] = {64, 1, C};
        return make_map_nd<3>(m, in + off, dims, strides, box);
    };
    const cuuint64_t sd[4] = {(cuuint64_t)p.dim, 2, (cuuint64_t)p.vdim, (cuuint64_t)c.n_chunks * p.heads};
    const cuuint64_t ss[3] = {(cuuint64_t)p.dim, (cuuint64_t)2 * p.dim, (cuuint64_t)2 * p.dim * p.vdim};
    const cuuint32_t sb[4] = {64, 1, VS, 1};
    if (!rows_map(&mq, p.q_off, p.dim) || !rows_map(&mk, p.k_off, p.dim) || !rows_map(&mv, p.v_off, p.vdim) || !make_map_nd<4>(&ms, c.state, sd, ss, sb))
        return cudaErrorInvalidValue;
    const bool rot = p.half > 0;
    const int slices = (p.vdim + VS - 1) / VS;
    const dim3 grid(c.n_chunks, p.heads, slices);
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
        return e != cudaSuccess ? e : launch_pdl(kernel, grid, dim3(THREADS), out_smem(p.dim), st, mq, mk, mv, ms, p, c);
    };
    return rot ? out(chunk_out_kernel<true>) : out(chunk_out_kernel<false>);
}

int bounds_status_linear_tc(bool reset);
LLM_DEFINE_BOUNDS_STATUS_READER(bounds_status_linear_tc)

}  // namespace llm
