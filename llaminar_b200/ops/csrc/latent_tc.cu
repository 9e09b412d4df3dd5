// Latent attention on the 5th-generation tensor cores: prompt chunks (latent_chunk_tc_kernel) and single rows
// (latent_rows_tc_kernel).  All operand tiles arrive by TMA in the 128-byte-swizzled form that the MMA reads.
// Every mbarrier wait is bounded; on a timeout the kernel raises the status word and tears down.
#include "latent.h"
#include "launch.h"
#include "tc_tile.cuh"

namespace llm {
namespace ltc {
using namespace tc5;


LLM_DEVICE int first_key(int pos, int window) { return window > 0 ? max(0, pos - window + 1) : 0; }
// ------------------------------------------------------------------------------------------------------------------------
// prompt chunks: 128 query rows of one head per CTA, keys in tiles of 128
//   S = Q K^T         M = 128 query rows, N = 128 keys, K = dim + rot; two accumulators
//   softmax           two threads per query row (= TMEM lane), 64 columns each; P goes back to TMEM as the A operand
//   O_tile = P V      M = 128, N = vdim, K = 128 keys; B is V^T (vdim rows of keys), which the value product writes directly
// The softmax threads keep the output row in registers and fold every O_tile in, scaled by the running-max correction.
// Warps 0-7 softmax, 8 TMA, 9 TMEM allocation and MMA issue.
// ------------------------------------------------------------------------------------------------------------------------
constexpr int BQ = 128, BK = 128, CHUNK_THREADS = 320;
enum Bar { K_FULL = 0, K_EMPTY = 2, V_FULL = 4, V_EMPTY = 6, S_FULL = 8, S_EMPTY = 10, P_FULL = 12, O_FULL = 13, O_EMPTY = 14, Q_FULL = 15, PAIR = 16, N_BARS = 20 };
constexpr int T_O = 256, T_P = 384;                // TMEM columns: S 0..255, O 256..383, P 384..447

template <int VD>
__global__ void __launch_bounds__(CHUNK_THREADS, 1) latent_chunk_tc_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_l,
                                                                           const __grid_constant__ CUtensorMap map_v, const LatentChunkParams p, int* status) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t s_bars[N_BARS];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort[2];
    // row maxima (and, at the end, sums) of a thread pair; an entry is overwritten only after the O_FULL wait of the tile, which
    // needs the partner's P_FULL arrival, which follows the partner's read
    __shared__ float s_xchg[2][BQ];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int head = blockIdx.y;
    const LatentSeq sq = p.seqs[blockIdx.z];
    const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * BQ;      // the last query tiles see the most keys: they go first
    if (q0 >= sq.q_len) return;                                      // uniform for the CTA, before any barrier or allocation
    if (sq.k_off % 8) {                                              // a TMA copy of the transposed values would start off a 16-byte boundary
        if (tid == 0 && status) atomicExch(status, (int)STATUS_BAD_ARG);
        return;
    }
    const int rows = min(BQ, sq.q_len - q0), pos0 = sq.q_pos0 + q0, pos_last = pos0 + rows - 1;
    const int tile0 = (max(first_key(pos0, p.window), sq.k_pos0) - sq.k_pos0) / BK;
    const int nt = (pos_last - sq.k_pos0) / BK + 1 - tile0;
    const int na = (p.dim + 63) / 64, nr = (p.rot + 63) / 64, nk = na + nr;       // operand atoms of a query or key row
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t sQ = base, sK = sQ + nk * ATOM, sV = sK + 2 * nk * ATOM;       // sV: [2 buffers][2 key halves]
    const uint32_t bars = smem_u32(s_bars);
    auto bar = [&](int i) { return bars + i * 8; };

    if (tid == 0) {
        s_abort[0] = 0; s_abort[1] = 0;
        const int counts[N_BARS] = {1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 8, 8, 8, 1, 8, 8, 2, 2, 2, 2};
        for (int i = 0; i < N_BARS; ++i) mbar_init(bar(i), counts[i]);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        fence_proxy_async();
    }
    if (warp == 9) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    volatile int* abort_flag = s_abort;

    if (warp < 8) {
        // queries: unrotated part copied, rotated part turned on the way
        const int un = p.dim / 8, ur = p.rot / 8;
        for (int i = tid; i < BQ * un; i += 256) {
            const int r = i / un, u = i % un;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (r < rows) v = *reinterpret_cast<const uint4*>(p.q + (size_t)(sq.q_start + q0 + r) * p.q_row + (size_t)head * p.q_head + u * 8);
            st_shared_v4(atom_addr(sQ + (u >> 3) * ATOM, r, u & 7), v);
        }
        for (int i = tid; i < BQ * ur; i += 256) {
            const int r = i / ur, u = i % ur;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (r < rows) {
                const size_t t = (size_t)sq.q_start + q0 + r;
                v = rotated8(p.q + t * p.q_row + (size_t)head * p.q_head + p.dim, u * 8, p.rot, p.angles + t * p.half, p.half);
            }
            st_shared_v4(atom_addr(sQ + (na + (u >> 3)) * ATOM, r, u & 7), v);
        }
        fence_proxy_async();
        __syncwarp();
        mbar_arrive_if(bar(Q_FULL), lane == 0);

        const int row = tid & 127, half = tid >> 7, q4 = warp & 3;
        const bool valid = row < rows;
        const int pos = pos0 + min(row, rows - 1);
        const int lim = pos + 1, low = first_key(pos, p.window);           // this row sees low <= key < lim
        const uint32_t t_lane = tmem + ((uint32_t)(q4 * 32) << 16);
        const float sl2 = p.scale * LOG2E;
        constexpr int HD = VD / 2;
        float o[HD];
#pragma unroll
        for (int i = 0; i < HD; ++i) o[i] = 0.f;
        float m = -INFINITY, l = 0.f, m_new = -INFINITY, mb = 0.f, alpha = 0.f, alpha_prev = 0.f;
        bool ok = true;
        int n_pair = 0;
        auto pair_meet = [&]() {                   // bounded rendezvous of the two warps that share these 32 rows
            __syncwarp();
            mbar_arrive_if(bar(PAIR + q4), lane == 0);
            const bool r = mbar_wait_warp(bar(PAIR + q4), n_pair & 1, abort_flag);
            ++n_pair;
            return r;
        };
        uint32_t ra[32], rb[32];
        // first pass over tile j: row maximum over this thread's 64 columns, exchanged with the partner thread
        auto pass1 = [&](int j) {
            if (!mbar_wait_warp(bar(S_FULL + (j & 1)), (j >> 1) & 1, abort_flag)) return false;
            tc_fence_after();
            const int key0 = sq.k_pos0 + (tile0 + j) * BK + half * 64;
            const uint32_t t_s = t_lane + (j & 1) * 128 + half * 64;
            tmem_ld32_issue(t_s, ra);
            tmem_ld32_issue(t_s + 32, rb);
            tmem_wait_ld(ra);
            tmem_wait_ld(rb);
            float mx = -INFINITY;
            if (key0 + 64 > lim || key0 < low) {
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    const int k0 = key0 + i, k1 = key0 + 32 + i;
                    mx = fmaxf(mx, k0 >= lim || k0 < low ? -INFINITY : __uint_as_float(ra[i]));
                    mx = fmaxf(mx, k1 >= lim || k1 < low ? -INFINITY : __uint_as_float(rb[i]));
                }
            } else {
#pragma unroll
                for (int i = 0; i < 32; ++i) mx = fmaxf(mx, fmaxf(__uint_as_float(ra[i]), __uint_as_float(rb[i])));
            }
            s_xchg[half][row] = mx;
            if (!pair_meet()) return false;
            mx = fmaxf(mx, s_xchg[half ^ 1][row]);
            m_new = fmaxf(m, mx * sl2);
            mb = m_new == -INFINITY ? 0.f : m_new;
            alpha = ex2(m - mb);
            return true;
        };
        // the tile's P V product is complete: fold it into the register copy of the output row
        auto fold = [&](int j) {
            if (!mbar_wait_warp(bar(O_FULL), j & 1, abort_flag)) return false;
            tc_fence_after();
            const uint32_t t_o = t_lane + T_O + half * HD;
            tmem_ld32_issue(t_o, ra);
            if constexpr (HD == 64) tmem_ld32_issue(t_o + 32, rb);
            tmem_wait_ld(ra);
            if constexpr (HD == 64) tmem_wait_ld(rb);
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                o[i] = o[i] * alpha_prev + __uint_as_float(ra[i]);
                if constexpr (HD == 64) o[32 + i] = o[32 + i] * alpha_prev + __uint_as_float(rb[i]);
            }
            tc_fence_before();
            __syncwarp();
            mbar_arrive_if(bar(O_EMPTY), lane == 0);
            return true;
        };
        for (int j = 0; j <= nt && ok; ++j) {
            if (j < nt) ok = pass1(j);
            if (ok && j > 0) ok = fold(j - 1);               // also frees P
            if (!ok || j == nt) break;
            const int key0 = sq.k_pos0 + (tile0 + j) * BK + half * 64;
            const bool need_mask = key0 + 64 > lim || key0 < low;
            const uint32_t t_s = t_lane + (j & 1) * 128 + half * 64;
            tmem_ld32_issue(t_s, ra);
            tmem_ld32_issue(t_s + 32, rb);
            tmem_wait_ld(ra);
            tmem_wait_ld(rb);
            float sum = 0.f;
            uint32_t w[32];
            auto probs_of = [&](int c, const uint32_t (&r)[32]) {
                if (need_mask) {
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        const int key = key0 + c * 32 + i;
                        const float p0 = key >= lim || key < low ? 0.f : ex2(__uint_as_float(r[i]) * sl2 - mb);
                        const float p1 = key + 1 >= lim || key + 1 < low ? 0.f : ex2(__uint_as_float(r[i + 1]) * sl2 - mb);
                        sum += p0 + p1;
                        w[c * 16 + (i >> 1)] = pack_bf16(p0, p1);
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        const float p0 = ex2(__uint_as_float(r[i]) * sl2 - mb), p1 = ex2(__uint_as_float(r[i + 1]) * sl2 - mb);
                        sum += p0 + p1;
                        w[c * 16 + (i >> 1)] = pack_bf16(p0, p1);
                    }
                }
            };
            probs_of(0, ra);
            probs_of(1, rb);
            tmem_st32(t_lane + T_P + half * 32, w);
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            mbar_arrive_if(bar(S_EMPTY + (j & 1)), lane == 0); mbar_arrive_if(bar(P_FULL), lane == 0);
            l = l * alpha + sum;
            m = m_new;
            alpha_prev = alpha;
        }
        if (ok) {                                  // the row's normaliser: both column halves, and the sink
            s_xchg[half][row] = l;
            ok = pair_meet();
        }
        if (ok && valid) {
            float lt = l + s_xchg[half ^ 1][row];
            if (p.sink) lt += exp2f(p.sink[head] * LOG2E - m);
            const float inv = 1.f / lt;
            __nv_bfloat16* dst = p.out + (size_t)(sq.q_start + q0 + row) * p.out_row + (size_t)head * p.vdim + half * HD;
#pragma unroll
            for (int u = 0; u < HD / 8; ++u) {
                if (half * HD + u * 8 >= p.vdim) break;
                if (p.gate) {
                    const uint4 g = *reinterpret_cast<const uint4*>(p.gate + (size_t)(sq.q_start + q0 + row) * p.gate_row + (size_t)head * p.vdim + half * HD + 8 * u);
                    const uint32_t gw[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        o[8 * u + 2 * i] *= __fdividef(1.f, 1.f + __expf(-bf16_lo(gw[i])));
                        o[8 * u + 2 * i + 1] *= __fdividef(1.f, 1.f + __expf(-bf16_hi(gw[i])));
                    }
                }
                *reinterpret_cast<uint4*>(dst + 8 * u) = make_uint4(pack_bf16(o[8 * u] * inv, o[8 * u + 1] * inv), pack_bf16(o[8 * u + 2] * inv, o[8 * u + 3] * inv),
                                                                    pack_bf16(o[8 * u + 4] * inv, o[8 * u + 5] * inv), pack_bf16(o[8 * u + 6] * inv, o[8 * u + 7] * inv));
            }
        }
    } else if (warp == 8) {
        if (elect_one()) {
            bool ok = true;
            for (int j = 0; j < nt && ok; ++j) {
                const int b = j & 1, key = sq.k_off + (tile0 + j) * BK;             // row of the key buffer
                ok = mbar_wait(bar(K_EMPTY + b), ((j >> 1) & 1) ^ 1, abort_flag);
                if (!ok) break;
                mbar_arrive_expect_tx(bar(K_FULL + b), nk * ATOM);
                for (int a = 0; a < na; ++a) tma_load_2d(sK + (b * nk + a) * ATOM, &map_k, head * p.dim + a * 64, key, bar(K_FULL + b));
                for (int a = 0; a < nr; ++a) tma_load_2d(sK + (b * nk + na + a) * ATOM, &map_l, p.rot_off + a * 64, key, bar(K_FULL + b));
                ok = mbar_wait(bar(V_EMPTY + b), ((j >> 1) & 1) ^ 1, abort_flag);
                if (!ok) break;
                mbar_arrive_expect_tx(bar(V_FULL + b), 2 * p.vdim * 128);
                for (int a = 0; a < 2; ++a) tma_load_2d(sV + (b * 2 + a) * ATOM, &map_v, key + a * 64, head * p.vdim, bar(V_FULL + b));
            }
        }
    } else if (elect_one()) {
        const uint32_t idesc_s = instr_desc(BK), idesc_o = instr_desc(p.vdim);
        bool ok = mbar_wait(bar(Q_FULL), 0, abort_flag);
        auto issue_s = [&](int j) {
            const int b = j & 1;
            ok = ok && mbar_wait(bar(K_FULL + b), (j >> 1) & 1, abort_flag) && mbar_wait(bar(S_EMPTY + b), ((j >> 1) & 1) ^ 1, abort_flag);
            if (!ok) return;
            tc_fence_after();
            uint32_t acc = 0;
            for (int a = 0; a < nk; ++a) {
                const int steps = (a < na ? min(64, p.dim - a * 64) : min(64, p.rot - (a - na) * 64)) / 16;
                const uint64_t qd = smem_desc_sw128(sQ + a * ATOM), kd = smem_desc_sw128(sK + (b * nk + a) * ATOM);
                for (int k = 0; k < steps; ++k) {
                    mma_f16(tmem + b * 128, qd + 2 * k, kd + 2 * k, idesc_s, acc);
                    acc = 1;
                }
            }
            mma_commit(bar(S_FULL + b));
            mma_commit(bar(K_EMPTY + b));
        };
        issue_s(0);
        for (int j = 0; j < nt && ok; ++j) {
            const int b = j & 1;
            if (j + 1 < nt) issue_s(j + 1);
            if (!ok) break;
            ok = mbar_wait(bar(P_FULL), j & 1, abort_flag) && mbar_wait(bar(V_FULL + b), (j >> 1) & 1, abort_flag) &&
                 mbar_wait(bar(O_EMPTY), (j & 1) ^ 1, abort_flag);
            if (!ok) break;
            tc_fence_after();
#pragma unroll
            for (int ks = 0; ks < 8; ++ks)          // 16 keys: 8 TMEM columns of P, 32 bytes of a V^T row
                mma_f16_ts(tmem + T_O, tmem + T_P + ks * 8, smem_desc_sw128(sV + (b * 2 + (ks >> 2)) * ATOM) + 2 * (ks & 3), idesc_o, ks > 0 ? 1u : 0u);
            mma_commit(bar(O_FULL));
            mma_commit(bar(V_EMPTY + b));
        }
    }
    tc_fence_before();
    __syncthreads();
    teardown(abort_flag, tid, status);
    if (warp == 9) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512) : "memory");
}

// ------------------------------------------------------------------------------------------------------------------------
// single rows: N heads of one row per CTA, keys in tiles of 64 (one page)
//   S = Q C^T         M = 128, N = 64 keys, K = latent + rotated part.  Q is the A operand in TMEM, its N rows (heads) repeated in
//                     every warp's lanes: each softmax warp finds all heads in its own lanes and takes 16 of the keys.  The cache
//                     rows are the B operand as they lie.
//   softmax           one thread per head and 16 keys: maxima and sums need no shuffles, only an exchange between the four warps
//   O^T += C^T P^T    M = 128 latent values, N heads, K = 64 keys: the same rows again, read as an MN-major A operand
// One copy of the cache rows serves both products.  The accumulator O^T stays in TMEM and is rescaled only when a running
// maximum rises by more than 2^RESCALE_STEP.
// Warps 0-3 softmax, 4 TMA, 5 TMEM allocation and MMA issue.
// ------------------------------------------------------------------------------------------------------------------------
constexpr int ROWS_THREADS = 192, PAGE = 64, SLOTS = 3, HALF = 64 * 128;      // HALF: an atom of 64 rows x 64 bf16
constexpr float RESCALE_STEP = 8.f;
enum RBar { R_FULL = 0, R_EMPTY = R_FULL + SLOTS, RS_FULL = R_EMPTY + SLOTS, RS_EMPTY, RP_FULL, RO_DONE, RQ_FULL, RQ_LAT, R_MEET, R_BARS };

// Shared memory: a ring of three key tiles (2 atoms per 128 latent values and one for the rotated part), then P.  The queries
// pass through the third tile's place on their way to TMEM.
static __host__ __device__ inline int tile_atoms(int latent) { return latent / 64 + 1; }
static __host__ __device__ inline size_t rows_smem(int n, int latent) { return (size_t)SLOTS * tile_atoms(latent) * HALF + n * 128 + 1024; }
static __host__ __device__ inline uint32_t pow2_cols(uint32_t n) { uint32_t c = 32; while (c < n) c *= 2; return c; }

template <int N>
__global__ void __launch_bounds__(ROWS_THREADS, 1) latent_rows_tc_kernel(const __grid_constant__ CUtensorMap map_kv, const __grid_constant__ CUtensorMap map_q,
                                                                        const LatentRowsParams p, int* status) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t s_bars[R_BARS];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort[2];
    __shared__ float s_red[2][4][32];              // [tile parity] per warp: maxima (and sums at the end) of its lanes' heads
    __shared__ __align__(16) float s_head[4][32];  // per warp: running maximum (or factor) of every head, for broadcast reads
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int NB = p.rot_off / 128;
    const uint32_t tile_bytes = tile_atoms(p.rot_off) * HALF;
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t sC = base, sQ = sC + 2 * tile_bytes, sP = sC + SLOTS * tile_bytes;
    // TMEM: S 64 columns, O^T N columns per block, Q one column per two values
    const uint32_t c_o = 64, c_q = c_o + NB * N, tmem_cols = pow2_cols(c_q + NB * 64 + 32);
    const uint32_t bars = smem_u32(s_bars);
    auto bar = [&](int i) { return bars + i * 8; };
    // no early trigger: while this kernel fills the shared memory of its SMs, the CTAs of the kernels behind it would gather on
    // the few others and stay there
    if (tid == 0) {
        s_abort[0] = 0; s_abort[1] = 0;
        for (int i = 0; i < R_BARS; ++i) mbar_init(bar(i), i == RP_FULL || i == RQ_FULL || i == RS_EMPTY || i == R_MEET ? 4 : 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        fence_proxy_async();
    }
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem, t_o = tmem + c_o;
    volatile int* abort_flag = s_abort;
    pdl_wait();

    const int hg = blockIdx.x, split = blockIdx.y, z = blockIdx.z;
    const int t = p.rows ? p.rows[z] : z;
    const int pos = p.positions[t], lo = first_key(pos, p.window);
    const int* btab = p.block_table + (size_t)LLM_CHECK_INDEX(p.seq_ids[t], p.n_seqs) * p.max_pages;
    const int page0 = lo / PAGE, page_last = pos / PAGE;
    const int n_tiles = page_last - page0 + 1, per = (n_tiles + gridDim.y - 1) / gridDim.y;
    const int j0 = split * per, nt = max(0, min(n_tiles, j0 + per) - j0);
    const size_t part = (((size_t)z * gridDim.x + hg) * gridDim.y + split) * N;

    if (nt == 0) {
        if (tid < N) *reinterpret_cast<float2*>(p.part_ml + (part + tid) * 2) = make_float2(-INFINITY, 0.f);
    } else if (warp < 4) {
        // query operand: the latent part arrives in shared memory by TMA and moves on to TMEM, the rotated part is turned here
        const int hl = lane & (N - 1), head = hg * N + hl;      // the head of this lane (its warps hold copies of the same heads)
        const uint32_t t_lane = (uint32_t)(warp * 32) << 16;
        bool ok = true;
        int n_meet = 0;
        auto meet = [&]() {                         // bounded rendezvous of the four softmax warps
            __syncwarp();
            mbar_arrive_if(bar(R_MEET), lane == 0);
            const bool r = mbar_wait_warp(bar(R_MEET), n_meet & 1, abort_flag);
            ++n_meet;
            return r;
        };
#pragma unroll
        for (int k = 0; k < N * 8 / 128; ++k) {
            const int r = (tid + k * 128) >> 3, u = tid & 7, h = hg * N + r;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (h < p.n_heads && u * 8 < p.rot_dim)
                v = rotated8(static_cast<const __nv_bfloat16*>(p.q) + (size_t)t * p.q_row + (size_t)h * p.q_head + p.q_rot_off, u * 8, p.rot_dim,
                             p.angles + (size_t)t * p.half, p.half);
            st_shared_v4(atom_addr(sQ + 2 * NB * N * 128, r, u), v);
        }
        ok = meet() && mbar_wait_warp(bar(RQ_LAT), 0, abort_flag);
        for (int a = 0; a <= 2 * NB && ok; ++a) {
            uint32_t w[32];
#pragma unroll
            for (int u = 0; u < 8; ++u)
                asm volatile("ld.shared.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(w[4 * u]), "=r"(w[4 * u + 1]), "=r"(w[4 * u + 2]), "=r"(w[4 * u + 3])
                             : "r"(atom_addr(sQ + a * N * 128, hl, u)));
            tmem_st32(tmem + c_q + a * 32 + t_lane, w);
        }
        tmem_wait_st();
        tc_fence_before();
        fence_proxy_async();                        // the third tile may overwrite the staged queries
        __syncwarp();
        mbar_arrive_if(bar(RQ_FULL), lane == 0);

        const float sl2 = p.scale * LOG2E;
        float l = 0.f, m = -INFINITY;               // l: this warp's keys' share of the head's sum
        auto broadcast = [&](float mine, float (&out)[N]) {      // lane c's value -> out[c] in every lane
            __syncwarp();
            s_head[warp][lane] = mine;
            __syncwarp();
#pragma unroll
            for (int c = 0; c < N; c += 4) {
                const float4 f = *reinterpret_cast<const float4*>(&s_head[warp][c]);
                out[c] = f.x; out[c + 1] = f.y; out[c + 2] = f.z; out[c + 3] = f.w;
            }
        };
        for (int j = 0; j < nt && ok; ++j) {
            ok = mbar_wait_warp(bar(RS_FULL), j & 1, abort_flag);
            if (!ok) break;
            tc_fence_after();
            float s[16];
            {
                uint32_t raw[16];
                tmem_ld_n<16>(tmem + warp * 16 + t_lane, raw);
                tc_fence_before();
                __syncwarp();
                mbar_arrive_if(bar(RS_EMPTY), lane == 0);       // the next tile's scores may be issued
                const int key0 = (page0 + j0 + j) * PAGE + warp * 16;
#pragma unroll
                for (int i = 0; i < 16; ++i) s[i] = key0 + i >= lo && key0 + i <= pos ? __uint_as_float(raw[i]) * sl2 : -INFINITY;
            }
            float mx = s[0];
#pragma unroll
            for (int i = 1; i < 16; ++i) mx = fmaxf(mx, s[i]);
            // (the reads of s_red two tiles ago precede the last tile's RS_EMPTY arrivals, without which this tile's S is not issued)
            float (&red4)[4][32] = s_red[j & 1];
            red4[warp][lane] = mx;
            ok = meet();
            if (!ok) break;
            const float mt = fmaxf(fmaxf(red4[0][lane], red4[1][lane]), fmaxf(red4[2][lane], red4[3][lane]));
            const bool raise = mt > m + RESCALE_STEP;           // also the first tile, where m is -inf
            const float factor = raise ? ex2(m - mt) : 1.f;
            if (raise) m = mt;
            float sum = 0.f;
            uint32_t w[8];
#pragma unroll
            for (int i = 0; i < 16; i += 2) {
                const float p0 = ex2(s[i] - m), p1 = ex2(s[i + 1] - m);
                sum += p0 + p1;
                w[i >> 1] = pack_bf16(p0, p1);
            }
            l = l * factor + sum;
            if (j > 0) {                                        // P and the accumulator are free
                ok = mbar_wait_warp(bar(RO_DONE), (j - 1) & 1, abort_flag);
                if (!ok) break;
                tc_fence_after();
            }
            if (__any_sync(0xffffffffu, raise) && j > 0) {      // the same in all four warps
                float f[N];
                uint32_t raw[N];
                broadcast(factor, f);
                for (int b = 0; b < NB; ++b) {
                    tmem_ld_n<N>(t_o + b * N + t_lane, raw);
#pragma unroll
                    for (int c = 0; c < N; ++c) raw[c] = __float_as_uint(__uint_as_float(raw[c]) * f[c]);
                    tmem_st_n<N>(t_o + b * N + t_lane, raw);
                }
                tmem_wait_st();
            }
            if (lane < N) {
                st_shared_v4(atom_addr(sP, lane, 2 * warp), make_uint4(w[0], w[1], w[2], w[3]));
                st_shared_v4(atom_addr(sP, lane, 2 * warp + 1), make_uint4(w[4], w[5], w[6], w[7]));
            }
            tc_fence_before();
            fence_proxy_async();
            __syncwarp();
            mbar_arrive_if(bar(RP_FULL), lane == 0);
        }
        // the last products are complete, so every warp has arrived with its P and is done with the maxima in s_red
        ok = ok && mbar_wait_warp(bar(RO_DONE), (nt - 1) & 1, abort_flag);
        if (ok) {
            s_red[0][warp][lane] = l;
            ok = meet();
        }
        if (ok) {
            tc_fence_after();
            float lt = s_red[0][0][lane] + s_red[0][1][lane] + s_red[0][2][lane] + s_red[0][3][lane];       // lane c: head c
            uint32_t raw[N];
            if (gridDim.y == 1) {
                const int h0 = hg * N;
                if (p.sink && head < p.n_heads) lt += exp2f(p.sink[head] * LOG2E - m);
                float inv[N];
                broadcast(1.f / lt, inv);
                for (int b = 0; b < NB; ++b) {
                    tmem_ld_n<N>(t_o + b * N + t_lane, raw);
                    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (size_t)z * p.out_row + b * 128 + tid;
#pragma unroll
                    for (int c = 0; c < N; ++c)
                        if (h0 + c < p.n_heads) out[(size_t)(h0 + c) * p.out_head] = __float2bfloat16(__uint_as_float(raw[c]) * inv[c]);
                }
            } else {
                for (int b = 0; b < NB; ++b) {
                    tmem_ld_n<N>(t_o + b * N + t_lane, raw);
                    float* out = p.part_o + part * p.rot_off + b * 128 + tid;
#pragma unroll
                    for (int c = 0; c < N; ++c) out[(size_t)c * p.rot_off] = __uint_as_float(raw[c]);
                }
                if (tid < N) *reinterpret_cast<float2*>(p.part_ml + (part + tid) * 2) = make_float2(m, lt);
            }
        }
    } else if (warp == 4) {
        if (elect_one()) {
            bool ok = true;
            mbar_arrive_expect_tx(bar(RQ_LAT), 2 * NB * N * 128);
            for (int a = 0; a < 2 * NB; ++a) tma_load_3d(sQ + a * N * 128, &map_q, a * 64, z, hg * N, bar(RQ_LAT));      // heads past the last: zeros
            for (int j = 0; j < nt; ++j) {
                const int r0 = LLM_CHECK_INDEX(btab[page0 + j0 + j], p.n_pages) * PAGE, slot = j % SLOTS;
                ok = mbar_wait(bar(R_EMPTY + slot), ((j / SLOTS) & 1) ^ 1, abort_flag) && (j != 2 || mbar_wait(bar(RQ_FULL), 0, abort_flag));
                if (!ok) break;
                mbar_arrive_expect_tx(bar(R_FULL + slot), tile_bytes);
                for (int a = 0; a <= 2 * NB; ++a) tma_load_2d(sC + slot * tile_bytes + a * HALF, &map_kv, a * 64, r0, bar(R_FULL + slot));
            }
        }
    } else {
        // The whole warp walks the pipeline and elects a lane only around each batch of MMAs: loop counters, slots and
        // descriptors then stay warp-uniform, which the issue rate depends on.
        constexpr uint32_t idesc_s = instr_desc(PAGE), idesc_o = instr_desc(N) | (1u << 15);         // bit 15: A is MN-major
        const uint32_t tm = __shfl_sync(0xffffffffu, tmem, 0);
        const int n = __shfl_sync(0xffffffffu, nt, 0), rot_steps = (p.width - p.rot_off) / 16;
        const uint64_t c_desc = smem_desc_sw128(sC), cm_desc = smem_desc_mn_sw128(sC, HALF), p_desc = smem_desc_sw128(sP);
        bool ok = mbar_wait_warp(bar(RQ_FULL), 0, abort_flag);
        int s_slot = 0, s_phase = 0, o_slot = 0;
        auto issue_s = [&](int j) {
            ok = mbar_wait_warp(bar(R_FULL + s_slot), s_phase, abort_flag) && (j == 0 || mbar_wait_warp(bar(RS_EMPTY), (j - 1) & 1, abort_flag));
            if (!ok) return;
            tc_fence_after();
            uint64_t c = c_desc + (uint32_t)(s_slot * (tile_bytes / 16));
            uint32_t q = tm + c_q;
            if (elect_one()) {
                uint32_t acc = 0;
                for (int b = 0; b < NB; ++b) {
#pragma unroll
                    for (int ks = 0; ks < 8; ++ks) {
                        mma_f16_ts(tm, q + ks * 8, c + (ks >> 2) * (HALF / 16) + 2 * (ks & 3), idesc_s, acc);
                        acc = 1;
                    }
                    q += 64;
                    c += 2 * (HALF / 16);
                }
                for (int ks = 0; ks < rot_steps; ++ks) mma_f16_ts(tm, q + ks * 8, c + 2 * ks, idesc_s, 1u);
                mma_commit(bar(RS_FULL));
            }
            __syncwarp();
            if (++s_slot == SLOTS) { s_slot = 0; s_phase ^= 1; }
        };
        if (ok) issue_s(0);
        for (int j = 0; j < n && ok; ++j) {
            if (j + 1 < n) issue_s(j + 1);
            ok = ok && mbar_wait_warp(bar(RP_FULL), j & 1, abort_flag);
            if (!ok) break;
            tc_fence_after();
            if (elect_one()) {
                uint64_t a = cm_desc + (uint32_t)(o_slot * (tile_bytes / 16));
                const uint32_t more = j > 0 ? 1u : 0u;
                for (int b = 0; b < NB; ++b) {
#pragma unroll
                    for (int ks = 0; ks < 4; ++ks)              // 16 keys: two groups of eight rows
                        mma_f16(tm + c_o + b * N, a + ks * (2048 / 16), p_desc + 2 * ks, idesc_o, ks > 0 ? 1u : more);
                    a += 2 * (HALF / 16);
                }
                mma_commit(bar(RO_DONE));
                mma_commit(bar(R_EMPTY + o_slot));
            }
            __syncwarp();
            if (++o_slot == SLOTS) o_slot = 0;
        }
    }
    tc_fence_before();
    __syncthreads();
    teardown(abort_flag, tid, status);
    if (warp == 5) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(tmem_cols) : "memory");
}

// ---- host side ---------------------------------------------------------------------------------------------------------
}  // namespace ltc

bool latent_chunk_tc_fits(int dim, int rot, int vdim) {
    const int nk = (dim + 63) / 64 + (rot + 63) / 64;
    return dim % 16 == 0 && rot % 16 == 0 && vdim % 16 == 0 && dim > 0 && rot > 0 && vdim >= 16 && vdim <= 128 && nk <= 3;
}

cudaError_t launch_latent_chunk_tc(const LatentChunkParams& p, int n_keys, int n_seqs, int max_q_len, int* status, cudaStream_t st) {
    using namespace ltc;
    if (!latent_chunk_tc_fits(p.dim, p.rot, p.vdim) || p.n_heads > 65535 || n_seqs > 65535 || n_keys % 8) return cudaErrorInvalidValue;
    CUtensorMap mk, ml, mv;
    if (!make_map(&mk, p.k, (uint64_t)p.n_heads * p.dim, n_keys, (uint64_t)p.n_heads * p.dim, 128) || !make_map(&ml, p.lat, p.lat_row, n_keys, p.lat_row, 128) ||
        !make_map(&mv, p.v, n_keys, (uint64_t)p.n_heads * p.vdim, n_keys, p.vdim))
        return cudaErrorInvalidValue;
    const int nk = (p.dim + 63) / 64 + (p.rot + 63) / 64;
    const size_t smem = (size_t)(3 * nk + 4) * ATOM + 1024;
    const dim3 grid((max_q_len + BQ - 1) / BQ, p.n_heads, n_seqs);
    auto go = [&](auto kernel) {
        cudaError_t e = raise_smem(kernel, smem);
        if (e != cudaSuccess) return e;
        kernel<<<grid, CHUNK_THREADS, smem, st>>>(mk, ml, mv, p, status);
        return cudaGetLastError();
    };
    return p.vdim <= 64 ? go(latent_chunk_tc_kernel<64>) : go(latent_chunk_tc_kernel<128>);
}

int latent_rows_tc_heads(int width, int rot_off, int rot_dim, int n_heads) {
    if (rot_off % 128 || rot_off < 128 || rot_off > 512 || width % 16 || width - rot_off > 64 || width <= rot_off || rot_dim <= 0) return 0;
    return n_heads <= 16 ? 16 : 32;
}

cudaError_t launch_latent_rows_tc(const LatentRowsParams& p, int rows, int n_splits, int* status, cudaStream_t st) {
    using namespace ltc;
    const int n = latent_rows_tc_heads(p.width, p.rot_off, p.rot_dim, p.n_heads);
    if (!n || rows > 65535 || p.ql_row % 8 || p.ql_head % 8) return cudaErrorInvalidValue;
    CUtensorMap m;
    if (!make_map(&m, p.kv, p.width, (uint64_t)p.n_pages * PAGE, p.width, PAGE)) return cudaErrorInvalidValue;
    CUtensorMap mq;                                          // [head][row][latent], boxes of 64 values x 1 row x n heads
    {
        const cuuint64_t dims[3] = {(cuuint64_t)p.rot_off, (cuuint64_t)rows, (cuuint64_t)p.n_heads}, strides[2] = {p.ql_row * 2, p.ql_head * 2};
        const cuuint32_t box[3] = {64, 1, (cuuint32_t)n}, estr[3] = {1, 1, 1};
        if (!encode_fn() || (reinterpret_cast<uintptr_t>(p.q_lat) & 15) ||
            encode_fn()(&mq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(p.q_lat), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                        CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
            return cudaErrorInvalidValue;
    }
    const size_t smem = rows_smem(n, p.rot_off);
    const dim3 grid((p.n_heads + n - 1) / n, n_splits, rows);
    auto go = [&](auto kernel) {
        cudaError_t e = raise_smem(kernel, smem);
        return e != cudaSuccess ? e : launch_pdl(kernel, grid, dim3(ROWS_THREADS), smem, st, m, mq, p, status);
    };
    return n == 16 ? go(latent_rows_tc_kernel<16>) : go(latent_rows_tc_kernel<32>);
}

int bounds_status_latent_tc(bool reset);
LLM_DEFINE_BOUNDS_STATUS_READER(bounds_status_latent_tc)

}  // namespace llm
