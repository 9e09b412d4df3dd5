// Attention over a low-rank latent cache.
//
// A token's cache row is [kv latent, kv_rank values padded to rot_off | rotated key part | padding to width]; pages hold 64 rows
// and all heads share them.  With per-head key matrix K_h and value matrix V_h the score of query q = [n | r] against key row
// [c | e] is n.(K_h c) + r.e = (K_h^T n).c + r.e, and the output of head h is V_h (sum p c).  Two forms of the same sum:
//
//   latent_rows    single rows (decode steps, one- or few-token portions): the query is moved into the latent space, so a key
//                  costs one cache row for all heads.  16 heads per CTA share the M dimension of the MMA; keys in tiles of 32
//                  through a cp.async ring; the key range is split over blockIdx.y and merged by a second kernel.
//   latent_chunk   prompt chunks: keys and values are written out per head by a matrix product beforehand (cheaper per
//                  query row than the latent form), 128 query rows per CTA, keys in tiles of 64.
//   latent_plain   one row and head per CTA in float arithmetic: the 32-bit mode, and sizes the kernels above do not take.
//
// All take a sliding window (row i sees j with i - window < j <= i) and a per-head sink logit, which joins the softmax
// denominator once, with no value.
#include "common.cuh"
#include "latent.h"
#include "launch.h"

namespace llm {

namespace {

constexpr int PAGE = 64;
constexpr float LOG2E = 1.4426950408889634f;

LLM_DEVICE float to_f(float v) { return v; }
LLM_DEVICE float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <class T> LLM_DEVICE T from_f(float v);
template <> LLM_DEVICE float from_f<float>(float v) { return v; }
template <> LLM_DEVICE __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

LLM_DEVICE void cp_async16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src));
}
LLM_DEVICE void cp_async_commit() { asm volatile("cp.async.commit_group;"); }
template <int N> LLM_DEVICE void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N)); }
LLM_DEVICE void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
LLM_DEVICE void ldsm_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
LLM_DEVICE void ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
LLM_DEVICE void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
LLM_DEVICE float quad_max(float v) {
    v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
    return fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
}
LLM_DEVICE float quad_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    return v + __shfl_xor_sync(0xffffffffu, v, 2);
}

// value i of a rotated part of `rot_dim` values: pairs (i, i + half) turn, the rest passes
template <class T> LLM_DEVICE float rotated(const T* x, int i, const float2* ang, int half) {
    if (i < half) return to_f(x[i]) * ang[i].x - to_f(x[i + half]) * ang[i].y;
    if (i < 2 * half) return to_f(x[i]) * ang[i - half].x + to_f(x[i - half]) * ang[i - half].y;
    return to_f(x[i]);
}

// values i0 .. i0 + 7 of it, zero from `n` on (reads no value past n)
LLM_DEVICE uint4 rotated8(const __nv_bfloat16* x, int i0, int n, const float2* ang, int half) {
    float v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = i0 + j < n ? rotated(x, i0 + j, ang, half) : 0.f;
    return make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}

LLM_DEVICE int first_key(int pos, int window) { return window > 0 ? max(0, pos - window + 1) : 0; }

// ---- cache rows --------------------------------------------------------------------------------------------------------
template <class T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentPrepParams p) {
    __shared__ float red[2][4];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const T* d = static_cast<const T*>(p.down) + (size_t)t * p.down_stride;
    const int pos = p.positions[t], seq = LLM_CHECK_INDEX(p.seq_ids[t], p.n_seqs);
    const int page = LLM_CHECK_INDEX(p.block_table[(size_t)seq * p.max_pages + pos / PAGE], p.n_pages);
    T* row = static_cast<T*>(p.kv) + ((size_t)page * PAGE + pos % PAGE) * p.width;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < p.q_rank; i += 128) { const float v = to_f(d[i]); sq += v * v; }
    for (int i = threadIdx.x; i < p.kv_rank; i += 128) { const float v = to_f(d[p.q_rank + i]); sk += v * v; }
    sq = warp_sum(sq); sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sk; }
    __syncthreads();
    sq = red[0][0] + red[0][1] + red[0][2] + red[0][3];
    sk = red[1][0] + red[1][1] + red[1][2] + red[1][3];
    const float iq = 1.f / sqrtf(sq / (float)p.q_rank + p.eps), ik = 1.f / sqrtf(sk / (float)p.kv_rank + p.eps);
    T* cq = static_cast<T*>(p.cq) + (size_t)t * p.cq_stride;
    for (int i = threadIdx.x; i < (int)p.cq_stride; i += 128) cq[i] = from_f<T>(i < p.q_rank ? to_f(d[i]) * iq * p.q_norm[i] : 0.f);
    for (int i = threadIdx.x; i < p.width; i += 128) {
        float v = 0.f;
        if (i < p.kv_rank) v = to_f(d[p.q_rank + i]) * ik * p.kv_norm[i];
        else if (i >= p.rot_off && i < p.rot_off + p.rot_dim) v = rotated(d + p.q_rank + p.kv_rank, i - p.rot_off, p.angles + (size_t)t * p.half, p.half);
        row[i] = from_f<T>(v);
    }
}

// The bf16 form for sizes that are multiples of 8: a warp per token, which keeps the row in registers as 16-byte units.
constexpr int PREP_UNITS = 12, PREP_WARPS = 4;
template <int UNITS>
__global__ void __launch_bounds__(32 * PREP_WARPS) latent_prep_vec_kernel(const LatentPrepParams p, int rows) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, t = blockIdx.x * PREP_WARPS + (threadIdx.x >> 5);
    if (t >= rows) return;
    const __nv_bfloat16* d = static_cast<const __nv_bfloat16*>(p.down) + (size_t)t * p.down_stride;
    const int nq = p.q_rank / 8, n = nq + p.kv_rank / 8;
    uint4 w[UNITS];
#pragma unroll
    for (int i = 0; i < UNITS; ++i) {
        const int u = lane + i * 32;
        w[i] = u < n ? *reinterpret_cast<const uint4*>(d + u * 8) : make_uint4(0, 0, 0, 0);
    }
    const int pos = p.positions[t], seq = LLM_CHECK_INDEX(p.seq_ids[t], p.n_seqs);
    const int page = LLM_CHECK_INDEX(p.block_table[(size_t)seq * p.max_pages + pos / PAGE], p.n_pages);
    __nv_bfloat16* row = static_cast<__nv_bfloat16*>(p.kv) + ((size_t)page * PAGE + pos % PAGE) * p.width;
    for (int u = lane; u < (p.width - p.rot_off) / 8; u += 32)           // rotated part and padding
        *reinterpret_cast<uint4*>(row + p.rot_off + u * 8) = rotated8(d + p.q_rank + p.kv_rank, u * 8, p.rot_dim, p.angles + (size_t)t * p.half, p.half);
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int i = 0; i < UNITS; ++i) {
        const uint32_t x[4] = {w[i].x, w[i].y, w[i].z, w[i].w};
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) { const float a = bf16_lo(x[j]), b = bf16_hi(x[j]); ss += a * a + b * b; }
        if (lane + i * 32 < nq) sq += ss; else sk += ss;
    }
    sq = warp_sum(sq); sk = warp_sum(sk);
    const float iq = 1.f / sqrtf(sq / (float)p.q_rank + p.eps), ik = 1.f / sqrtf(sk / (float)p.kv_rank + p.eps);
#pragma unroll
    for (int i0 = 0; i0 < UNITS; i0 += 4) {                 // gains of four units in flight at a time
        float4 g[4][2];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int u = min(lane + (i0 + i) * 32, n - 1);
            const float4* gp = reinterpret_cast<const float4*>(u < nq ? p.q_norm + u * 8 : p.kv_norm + (u - nq) * 8);
            g[i][0] = gp[0];
            g[i][1] = gp[1];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int u = lane + (i0 + i) * 32;
            const uint4 x = w[i0 + i];
            const float inv = u < nq ? iq : ik;
            const float4 g0 = g[i][0], g1 = g[i][1];
            const uint4 o = make_uint4(pack_bf16(bf16_lo(x.x) * inv * g0.x, bf16_hi(x.x) * inv * g0.y), pack_bf16(bf16_lo(x.y) * inv * g0.z, bf16_hi(x.y) * inv * g0.w),
                                       pack_bf16(bf16_lo(x.z) * inv * g1.x, bf16_hi(x.z) * inv * g1.y), pack_bf16(bf16_lo(x.w) * inv * g1.z, bf16_hi(x.w) * inv * g1.w));
            if (u < n) *reinterpret_cast<uint4*>(u < nq ? static_cast<__nv_bfloat16*>(p.cq) + (size_t)t * p.cq_stride + u * 8 : row + (u - nq) * 8) = o;
        }
    }
}

// one warp per key row
template <class T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const T* kv, const LatentSeq* seqs, const int* block_table, int max_pages, int n_pages,
                                                            int width, T* out) {
    const LatentSeq s = seqs[blockIdx.y];
    const int i = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (i >= (s.k_len + 7) / 8 * 8) return;
    if (i >= s.k_len) {                     // the next sequence's rows start at a multiple of 8: zeros in between
        uint4* dst = reinterpret_cast<uint4*>(out + (size_t)(s.k_off + i) * width);
        for (int u = threadIdx.x & 31; u < width * (int)sizeof(T) / 16; u += 32) dst[u] = make_uint4(0, 0, 0, 0);
        return;
    }
    const int pos = s.k_pos0 + i;
    const int page = LLM_CHECK_INDEX(block_table[(size_t)s.seq * max_pages + pos / PAGE], n_pages);
    const uint4* src = reinterpret_cast<const uint4*>(kv + ((size_t)page * PAGE + pos % PAGE) * width);
    uint4* dst = reinterpret_cast<uint4*>(out + (size_t)(s.k_off + i) * width);
    for (int u = threadIdx.x & 31; u < width * (int)sizeof(T) / 16; u += 32) dst[u] = src[u];
}

// ---- single rows, any size, float arithmetic -----------------------------------------------------------------------------
template <class T>
__global__ void __launch_bounds__(128) latent_plain_kernel(const LatentRowsParams p) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_score[64];
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, z = blockIdx.y, t = p.rows ? p.rows[z] : z;
    float *sq = sm, *so = sm + p.width;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, R = p.rot_off;
    const int pos = p.positions[t];
    const int* btab = p.block_table + (size_t)LLM_CHECK_INDEX(p.seq_ids[t], p.n_seqs) * p.max_pages;
    const T* ql = static_cast<const T*>(p.q_lat) + (size_t)z * p.ql_row + (size_t)h * p.ql_head;
    const T* qr = static_cast<const T*>(p.q) + (size_t)t * p.q_row + (size_t)h * p.q_head + p.q_rot_off;
    for (int i = threadIdx.x; i < p.width; i += 128) {
        float v = 0.f;
        if (i < R) v = to_f(ql[i]);
        else if (i < R + p.rot_dim) v = to_f(from_f<T>(rotated(qr, i - R, p.angles + (size_t)t * p.half, p.half)));
        sq[i] = v;
    }
    for (int i = threadIdx.x; i < R; i += 128) so[i] = 0.f;
    __syncthreads();
    float m = p.sink ? p.sink[h] : -INFINITY, l = p.sink ? 1.f : 0.f;
    for (int k0 = first_key(pos, p.window); k0 <= pos; k0 += 64) {
        const int n = min(64, pos + 1 - k0);
        for (int j = warp; j < n; j += 4) {
            const int key = k0 + j, page = LLM_CHECK_INDEX(btab[key / PAGE], p.n_pages);
            const T* row = static_cast<const T*>(p.kv) + ((size_t)page * PAGE + key % PAGE) * p.width;
            float s = 0.f;
            for (int i = lane; i < R + p.rot_dim; i += 32) s = fmaf(sq[i], to_f(row[i]), s);
            s = warp_sum(s);
            if (lane == 0) s_score[j] = s * p.scale;
        }
        __syncthreads();
        float nm = m;
        for (int j = 0; j < n; ++j) nm = fmaxf(nm, s_score[j]);
        const float c = expf(m - nm);
        __syncthreads();
        if ((int)threadIdx.x < n) s_score[threadIdx.x] = expf(s_score[threadIdx.x] - nm);
        __syncthreads();
        float ps = 0.f;
        for (int j = 0; j < n; ++j) ps += s_score[j];
        l = l * c + ps;
        m = nm;
        for (int i = threadIdx.x; i < R; i += 128) {
            float a = so[i] * c;
            for (int j = 0; j < n; ++j) {
                const int key = k0 + j, page = LLM_CHECK_INDEX(btab[key / PAGE], p.n_pages);
                a = fmaf(s_score[j], to_f(static_cast<const T*>(p.kv)[((size_t)page * PAGE + key % PAGE) * p.width + i]), a);
            }
            so[i] = a;
        }
        __syncthreads();
    }
    T* o = static_cast<T*>(p.out) + (size_t)z * p.out_row + (size_t)h * p.out_head;
    for (int i = threadIdx.x; i < R; i += 128) o[i] = from_f<T>(so[i] / l);
}

// ---- single rows on the tensor cores ---------------------------------------------------------------------------------------
constexpr int KT = 32;               // keys per tile: half a page
__host__ __device__ inline int row_stride(int width) { return width + 8; }      // elements; odd number of 16-byte units
inline size_t rows_smem(int width, int stages) {
    return ((size_t)stages * KT + 16) * row_stride(width) * 2 + 16 * (KT + 8) * 2 + 4 * 16 * 4 * 2;
}

template <int NT, int STAGES>
__global__ void __launch_bounds__(128) latent_rows_kernel(const LatentRowsParams p) {
    extern __shared__ __align__(128) uint8_t smem[];
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int hg = blockIdx.x, split = blockIdx.y, z = blockIdx.z;
    const int t = p.rows ? p.rows[z] : z;
    const int LD = row_stride(p.width), R = p.rot_off, KS = p.width / 16;
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(smem);                 // [16][LD]
    __nv_bfloat16* sp = sq + 16 * LD;                                           // [16][KT + 8]
    float* s_max = reinterpret_cast<float*>(sp + 16 * (KT + 8));                // [4][16]
    float* s_sum = s_max + 64;                                                  // [4][16]
    __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(s_sum + 64);           // [STAGES][KT][LD]
    const uint32_t q_base = smem_u32(sq), p_base = smem_u32(sp), k_base = smem_u32(sk);

    const int pos = p.positions[t], lo = first_key(pos, p.window);
    const int* btab = p.block_table + (size_t)LLM_CHECK_INDEX(p.seq_ids[t], p.n_seqs) * p.max_pages;
    const int tile0 = lo / KT, n_tiles = pos / KT - tile0 + 1;
    const int per = (n_tiles + gridDim.y - 1) / gridDim.y;
    const int kt0 = tile0 + split * per, kt1 = min(tile0 + n_tiles, kt0 + per);

    auto issue = [&](int kt, int stage) {
        if (kt < kt1) {
            const int page = LLM_CHECK_INDEX(btab[kt * KT / PAGE], p.n_pages);
            const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.kv) + ((size_t)page * PAGE + (kt * KT) % PAGE) * p.width;
            const uint32_t dst = k_base + stage * KT * LD * 2;
            // the tile is one contiguous run of 16-byte units; row = unit / upr by multiplication (exact: units < 2^20 / upr)
            const unsigned upr = p.width / 8, inv = (1u << 20) / upr + 1;
            for (unsigned u = threadIdx.x; u < KT * upr; u += 128) {
                const unsigned r = (u * inv) >> 20;
                cp_async16(dst + (r * LD + (u - r * upr) * 8) * 2, src + (size_t)u * 8);
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) issue(kt0 + s, s);

    // queries of the 16 heads: latent part, rotated part, zero padding (and zero rows past the last head)
    for (int i = threadIdx.x; i < 16 * (LD / 8); i += 128) {
        const int r = i / (LD / 8), u = i % (LD / 8), h = hg * 16 + r;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (h < p.n_heads) {
            if (u * 8 < R) v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.q_lat) + (size_t)z * p.ql_row + (size_t)h * p.ql_head + u * 8);
            else v = rotated8(static_cast<const __nv_bfloat16*>(p.q) + (size_t)t * p.q_row + (size_t)h * p.q_head + p.q_rot_off, u * 8 - R, p.rot_dim,
                              p.angles + (size_t)t * p.half, p.half);
        }
        *reinterpret_cast<uint4*>(sq + r * LD + u * 8) = v;
    }

    float o[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[n][i] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    const float sl2 = p.scale * LOG2E;
    const int i0 = lane >> 2, i1 = i0 + 8, mat = lane >> 3, r8 = lane & 7;
    const int col_base = warp * NT * 8;

    for (int kt = kt0; kt < kt1; ++kt) {
        const int stage = (kt - kt0) % STAGES;
        cp_async_wait<STAGES - 2>();
        __syncthreads();
        issue(kt + STAGES - 1, (kt - kt0 + STAGES - 1) % STAGES);
        const uint32_t kb = k_base + stage * KT * LD * 2;
        // this warp's 8 keys
        float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
        const uint32_t kaddr = kb + ((warp * 8 + r8) * LD + mat * 8) * 2;
        const uint32_t qaddr = q_base + ((lane & 15) * LD + (lane >> 4) * 8) * 2;
        int ks = 0;
#pragma unroll 4
        for (; ks + 1 < KS; ks += 2) {
            uint32_t b[4], a0[4], a1[4];
            ldsm_x4(kaddr + ks * 32, b);
            ldsm_x4(qaddr + ks * 32, a0);
            ldsm_x4(qaddr + ks * 32 + 32, a1);
            mma_bf16(s, a0, b[0], b[1]);
            mma_bf16(s2, a1, b[2], b[3]);
        }
        if (ks < KS) {
            uint32_t b0, b1, a0[4];
            ldsm_x2(kb + ((warp * 8 + r8) * LD + (mat & 1) * 8) * 2 + ks * 32, b0, b1);
            ldsm_x4(qaddr + ks * 32, a0);
            mma_bf16(s, a0, b0, b1);
        }
        const int key0 = kt * KT + warp * 8 + (lane & 3) * 2;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const bool seen = key0 + e >= lo && key0 + e <= pos;
            s[e] = seen ? (s[e] + s2[e]) * sl2 : -INFINITY;
            s[2 + e] = seen ? (s[2 + e] + s2[2 + e]) * sl2 : -INFINITY;
        }
        const float mx0 = quad_max(fmaxf(s[0], s[1])), mx1 = quad_max(fmaxf(s[2], s[3]));
        if ((lane & 3) == 0) { s_max[warp * 16 + i0] = mx0; s_max[warp * 16 + i1] = mx1; }
        __syncthreads();
        float nm0 = m0, nm1 = m1;
#pragma unroll
        for (int w = 0; w < 4; ++w) { nm0 = fmaxf(nm0, s_max[w * 16 + i0]); nm1 = fmaxf(nm1, s_max[w * 16 + i1]); }
        // every tile of the range holds at least one key that the row sees, so the maxima are finite
        const float c0 = exp2f(m0 - nm0), c1 = exp2f(m1 - nm1);
        m0 = nm0; m1 = nm1;
#pragma unroll
        for (int e = 0; e < 2; ++e) { s[e] = exp2f(s[e] - nm0); s[2 + e] = exp2f(s[2 + e] - nm1); }
        l0 = l0 * c0 + s[0] + s[1];
        l1 = l1 * c1 + s[2] + s[3];
        *reinterpret_cast<uint32_t*>(sp + i0 * (KT + 8) + warp * 8 + (lane & 3) * 2) = pack_bf16(s[0], s[1]);
        *reinterpret_cast<uint32_t*>(sp + i1 * (KT + 8) + warp * 8 + (lane & 3) * 2) = pack_bf16(s[2], s[3]);
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[n][0] *= c0; o[n][1] *= c0; o[n][2] *= c1; o[n][3] *= c1; }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < KT / 16; ++kk) {
            uint32_t a[4];
            ldsm_x4(p_base + ((lane & 15) * (KT + 8) + kk * 16 + (lane >> 4) * 8) * 2, a);
            const uint32_t vaddr = kb + ((kk * 16 + (mat & 1) * 8 + r8) * LD + col_base + (mat >> 1) * 8) * 2;
#pragma unroll
            for (int c = 0; c < NT / 2; ++c) {
                if (col_base + c * 16 < R) {                       // the same for all lanes of the warp
                    uint32_t b[4];
                    ldsm_x4_t(vaddr + c * 32, b);
                    mma_bf16(o[2 * c], a, b[0], b[1]);
                    mma_bf16(o[2 * c + 1], a, b[2], b[3]);
                }
            }
        }
    }
    cp_async_wait<0>();
    l0 = quad_sum(l0); l1 = quad_sum(l1);
    if ((lane & 3) == 0) { s_sum[warp * 16 + i0] = l0; s_sum[warp * 16 + i1] = l1; }
    __syncthreads();
    l0 = s_sum[i0] + s_sum[16 + i0] + s_sum[32 + i0] + s_sum[48 + i0];
    l1 = s_sum[i1] + s_sum[16 + i1] + s_sum[32 + i1] + s_sum[48 + i1];
    if (gridDim.y == 1) {
        auto finish = [&](int i, float m, float l) -> float {      // 1 / denominator relative to m
            const int h = hg * 16 + i;
            if (p.sink && h < p.n_heads) {
                // exp2(sink - m) overflows only if the sink outweighs every key by 2^127: the quotient is then zero, as it should
                l += exp2f(p.sink[h] * LOG2E - m);
            }
            return 1.f / l;
        };
        const float v0 = finish(i0, m0, l0), v1 = finish(i1, m1, l1);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            const int col = col_base + n * 8 + (lane & 3) * 2;
            if (col >= R) continue;
            __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (size_t)z * p.out_row + col;
            if (hg * 16 + i0 < p.n_heads) *reinterpret_cast<uint32_t*>(out + (size_t)(hg * 16 + i0) * p.out_head) = pack_bf16(o[n][0] * v0, o[n][1] * v0);
            if (hg * 16 + i1 < p.n_heads) *reinterpret_cast<uint32_t*>(out + (size_t)(hg * 16 + i1) * p.out_head) = pack_bf16(o[n][2] * v1, o[n][3] * v1);
        }
        return;
    }
    const size_t part = (((size_t)z * gridDim.x + hg) * gridDim.y + split) * 16;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
        const int col = col_base + n * 8 + (lane & 3) * 2;
        if (col >= R) continue;
        *reinterpret_cast<float2*>(p.part_o + (part + i0) * R + col) = make_float2(o[n][0], o[n][1]);
        *reinterpret_cast<float2*>(p.part_o + (part + i1) * R + col) = make_float2(o[n][2], o[n][3]);
    }
    if (warp == 0 && (lane & 3) == 0) {
        *reinterpret_cast<float2*>(p.part_ml + (part + i0) * 2) = make_float2(m0, l0);
        *reinterpret_cast<float2*>(p.part_ml + (part + i1) * 2) = make_float2(m1, l1);
    }
}

constexpr int MAX_SPLITS = 64;
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentRowsParams p, int n_splits, int groups, int group) {
    __shared__ float s_w[MAX_SPLITS];
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, z = blockIdx.y, R = p.rot_off, lane = threadIdx.x & 31;
    const size_t part = ((size_t)z * groups + h / group) * n_splits * group + h % group;
    if (threadIdx.x < 32) {
        const float2 none = make_float2(-INFINITY, 0.f);
        const float2 a = lane < n_splits ? *reinterpret_cast<const float2*>(p.part_ml + (part + (size_t)lane * group) * 2) : none;
        const float2 b = lane + 32 < n_splits ? *reinterpret_cast<const float2*>(p.part_ml + (part + (size_t)(lane + 32) * group) * 2) : none;
        const float sink = p.sink ? p.sink[h] * LOG2E : -INFINITY;
        const float m = fmaxf(warp_max(fmaxf(a.x, b.x)), sink);
        const float wa = exp2f(a.x - m), wb = exp2f(b.x - m);               // 0 for a split without keys
        const float inv = 1.f / (warp_sum(wa * a.y + wb * b.y) + exp2f(sink - m));
        s_w[lane] = wa * inv;
        s_w[lane + 32] = wb * inv;
    }
    __syncthreads();
    for (int c = threadIdx.x * 4; c < R; c += 512) {
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int s = 0; s < n_splits; ++s) {
            const float w = s_w[s];
            if (w == 0.f) continue;                                         // a split without keys wrote no sums
            const float4 v = *reinterpret_cast<const float4*>(p.part_o + (part + (size_t)s * group) * R + c);
            a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
        }
        *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p.out) + (size_t)z * p.out_row + (size_t)h * p.out_head + c) =
            make_uint2(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w));
    }
}

// ---- prompt chunks on the tensor cores ---------------------------------------------------------------------------------------
constexpr int BQ = 128, BK = 64;

template <int DK, int DV>
constexpr size_t chunk_smem() { return ((size_t)BQ * (DK + 8) + 2 * BK * ((DK + 8) + (DV + 8))) * 2; }

template <int DK, int DV>
__global__ void __launch_bounds__(256) latent_chunk_kernel(const LatentChunkParams p) {
    extern __shared__ __align__(128) uint8_t smem[];
    const LatentSeq sq = p.seqs[blockIdx.z];
    // later rows see more keys (until the window fills): start them first
    const int qt0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * BQ;
    if (qt0 >= sq.q_len) return;
    const int head = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    constexpr int LQ = DK + 8, LK = DK + 8, LV = DV + 8;
    __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(smem);        // [BQ][LQ]
    __nv_bfloat16* s_kv = s_q + BQ * LQ;                                // [2][BK][LK] then [2][BK][LV]
    const uint32_t q_base = smem_u32(s_q), k_base = smem_u32(s_kv), v_base = k_base + 2 * BK * LK * 2;
    const int pos0 = sq.q_pos0 + qt0, n_rows = min(BQ, sq.q_len - qt0), pos_last = pos0 + n_rows - 1;
    const int key_lo = max(first_key(pos0, p.window), sq.k_pos0), key_hi = pos_last;          // positions
    const int b_lo = key_lo - sq.k_pos0, b_hi = key_hi - sq.k_pos0;                           // rows of the key buffer
    const int tile0 = b_lo / BK, tile1 = b_hi / BK + 1;

    // columns that no copy writes: padding of the head sizes up to the template's
    if (p.dim + p.rot < DK || p.vdim < DV) {
        for (int i = threadIdx.x; i < 2 * BK * (DK + 8 + DV + 8) / 2; i += 256) reinterpret_cast<uint32_t*>(s_kv)[i] = 0u;
        __syncthreads();
    }
    const int uk = p.dim / 8, ur = p.rot / 8, uv = p.vdim / 8;
    auto issue = [&](int tile, int stage) {
        if (tile < tile1) {
            const uint32_t kd = k_base + stage * BK * LK * 2, vd = v_base + stage * BK * LV * 2;
            // a quarter of a warp per key row: 8 lanes copy 128 contiguous bytes at a time
            for (int r = threadIdx.x >> 3; r < BK; r += 32) {
                const size_t row = (size_t)(sq.k_off + min(tile * BK + r, sq.k_len - 1));
                const __nv_bfloat16 *ks = p.k + (row * p.n_heads + head) * p.dim, *vs = p.v + (row * p.n_heads + head) * p.vdim;
                for (int u = threadIdx.x & 7; u < uk; u += 8) cp_async16(kd + (r * LK + u * 8) * 2, ks + u * 8);
                for (int u = threadIdx.x & 7; u < ur; u += 8) cp_async16(kd + (r * LK + p.dim + u * 8) * 2, p.lat + row * p.lat_row + p.rot_off + u * 8);
                for (int u = threadIdx.x & 7; u < uv; u += 8) cp_async16(vd + (r * LV + u * 8) * 2, vs + u * 8);
            }
        }
        cp_async_commit();
    };
    issue(tile0, 0);
    {   // queries: unrotated part as it is, rotated part turned here
        for (int r = warp; r < BQ; r += 8) {
            const bool live = r < n_rows;
            const size_t t = (size_t)sq.q_start + qt0 + (live ? r : 0);
            const __nv_bfloat16* src = p.q + t * p.q_row + (size_t)head * p.q_head;
            for (int u = lane; u < uk; u += 32)
                *reinterpret_cast<uint4*>(s_q + r * LQ + u * 8) = live ? *reinterpret_cast<const uint4*>(src + u * 8) : make_uint4(0, 0, 0, 0);
            for (int u = lane; u < LQ / 8 - uk; u += 32)
                *reinterpret_cast<uint4*>(s_q + r * LQ + p.dim + u * 8) = live ? rotated8(src + p.dim, u * 8, p.rot, p.angles + t * p.half, p.half) : make_uint4(0, 0, 0, 0);
        }
    }
    float o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[n][i] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    const float sl2 = p.scale * LOG2E;
    const int i0 = warp * 16 + (lane >> 2), i1 = i0 + 8, mat = lane >> 3, r8 = lane & 7;
    const int p0 = pos0 + i0, p1 = pos0 + i1;                         // rows past the chunk's end compute on zero queries
    const int lo0 = first_key(p0, p.window), lo1 = first_key(p1, p.window);
    const int w_first = pos0 + warp * 16, w_last = w_first + 15;      // positions of this warp's rows
    const int w_lo = first_key(w_first, p.window);

    for (int tile = tile0; tile < tile1; ++tile) {
        const int stage = (tile - tile0) & 1;
        cp_async_wait<0>();
        __syncthreads();
        issue(tile + 1, stage ^ 1);
        const int key_base = sq.k_pos0 + tile * BK;                   // position of the tile's first key
        if (key_base > w_last || key_base + BK <= w_lo) continue;     // nothing here for this warp
        const uint32_t kb = k_base + stage * BK * LK * 2, vb = v_base + stage * BK * LV * 2;
        float s[BK / 8][4];
#pragma unroll
        for (int n = 0; n < BK / 8; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) s[n][i] = 0.f;
        const uint32_t qaddr = q_base + ((warp * 16 + (lane & 15)) * LQ + (lane >> 4) * 8) * 2;
        const uint32_t kaddr = kb + (((mat >> 1) * 8 + r8) * LK + (mat & 1) * 8) * 2;
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
            uint32_t a[4];
            ldsm_x4(qaddr + ks * 32, a);
#pragma unroll
            for (int nb = 0; nb < BK / 16; ++nb) {
                uint32_t b[4];
                ldsm_x4(kaddr + nb * 16 * LK * 2 + ks * 32, b);
                mma_bf16(s[2 * nb], a, b[0], b[1]);
                mma_bf16(s[2 * nb + 1], a, b[2], b[3]);
            }
        }
        const bool need_mask = key_base + BK - 1 > w_first || (p.window > 0 && key_base < first_key(w_last, p.window));
        float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
        for (int n = 0; n < BK / 8; ++n) {
            const int key = key_base + n * 8 + (lane & 3) * 2;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                s[n][e] = (!need_mask || (key + e <= p0 && key + e >= lo0)) ? s[n][e] * sl2 : -INFINITY;
                s[n][2 + e] = (!need_mask || (key + e <= p1 && key + e >= lo1)) ? s[n][2 + e] * sl2 : -INFINITY;
                mx0 = fmaxf(mx0, s[n][e]);
                mx1 = fmaxf(mx1, s[n][2 + e]);
            }
        }
        const float nm0 = fmaxf(m0, quad_max(mx0)), nm1 = fmaxf(m1, quad_max(mx1));
        const float b0 = nm0 == -INFINITY ? 0.f : nm0, b1 = nm1 == -INFINITY ? 0.f : nm1;
        const float c0 = exp2f(m0 - b0), c1 = exp2f(m1 - b1);
        m0 = nm0; m1 = nm1;
        float ps0 = 0.f, ps1 = 0.f;
#pragma unroll
        for (int n = 0; n < BK / 8; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                s[n][e] = exp2f(s[n][e] - b0); ps0 += s[n][e];
                s[n][2 + e] = exp2f(s[n][2 + e] - b1); ps1 += s[n][2 + e];
            }
        l0 = l0 * c0 + ps0; l1 = l1 * c1 + ps1;
#pragma unroll
        for (int n = 0; n < DV / 8; ++n) { o[n][0] *= c0; o[n][1] *= c0; o[n][2] *= c1; o[n][3] *= c1; }
        const uint32_t vaddr = vb + (((mat & 1) * 8 + r8) * LV + (mat >> 1) * 8) * 2;
#pragma unroll
        for (int kk = 0; kk < BK / 16; ++kk) {
            const uint32_t a[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]), pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                                   pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]), pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
            for (int c = 0; c < DV / 16; ++c) {
                uint32_t b[4];
                ldsm_x4_t(vaddr + kk * 16 * LV * 2 + c * 32, b);
                mma_bf16(o[2 * c], a, b[0], b[1]);
                mma_bf16(o[2 * c + 1], a, b[2], b[3]);
            }
        }
    }
    cp_async_wait<0>();
    l0 = quad_sum(l0); l1 = quad_sum(l1);
    if (p.sink) {
        const float sk = p.sink[head] * LOG2E;
        l0 += exp2f(sk - m0);
        l1 += exp2f(sk - m1);
    }
    const float v0 = 1.f / l0, v1 = 1.f / l1;
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) {
        const int col = n * 8 + (lane & 3) * 2;
        if (col >= p.vdim) continue;
        auto store = [&](int i, float a, float b) {
            if (i >= n_rows) return;
            const size_t t = (size_t)sq.q_start + qt0 + i;
            if (p.gate) {
                const uint32_t g = *reinterpret_cast<const uint32_t*>(p.gate + t * p.gate_row + (size_t)head * p.vdim + col);
                a *= 1.f / (1.f + __expf(-bf16_lo(g)));
                b *= 1.f / (1.f + __expf(-bf16_hi(g)));
            }
            *reinterpret_cast<uint32_t*>(p.out + t * p.out_row + (size_t)head * p.vdim + col) = pack_bf16(a, b);
        };
        store(i0, o[n][0] * v0, o[n][1] * v0);
        store(i1, o[n][2] * v1, o[n][3] * v1);
    }
}

template <class K> cudaError_t raise_smem(K kernel, size_t bytes) {
    return bytes <= 48 * 1024 ? cudaSuccess : cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

}  // namespace

cudaError_t launch_latent_prep(const LatentPrepParams& p, int rows, bool f32, cudaStream_t st) {
    if (f32) return launch_pdl(latent_prep_kernel<float>, dim3(rows), dim3(128), 0, st, p);
    const bool vec = p.q_rank % 8 == 0 && p.kv_rank % 8 == 0 && p.rot_dim % 8 == 0 && p.down_stride % 8 == 0 && (int)p.cq_stride == p.q_rank &&
                     p.rot_off == p.kv_rank && (p.q_rank + p.kv_rank) / 8 <= PREP_UNITS * 32 &&
                     !((reinterpret_cast<uintptr_t>(p.down) | reinterpret_cast<uintptr_t>(p.q_norm) | reinterpret_cast<uintptr_t>(p.kv_norm)) & 15);
    if (vec) {
        const dim3 grid((rows + PREP_WARPS - 1) / PREP_WARPS), block(32 * PREP_WARPS);
        const int units = (p.q_rank + p.kv_rank) / 8;
        if (units <= 4 * 32) return launch_pdl(latent_prep_vec_kernel<4>, grid, block, 0, st, p, rows);
        if (units <= 8 * 32) return launch_pdl(latent_prep_vec_kernel<8>, grid, block, 0, st, p, rows);
        return launch_pdl(latent_prep_vec_kernel<PREP_UNITS>, grid, block, 0, st, p, rows);
    }
    return launch_pdl(latent_prep_kernel<__nv_bfloat16>, dim3(rows), dim3(128), 0, st, p);
}

cudaError_t launch_latent_gather(const void* kv, const LatentSeq* seqs, int n, int max_k_len, const int* block_table, int max_pages,
                                 int n_pages, int width, void* out, bool f32, cudaStream_t st) {
    const dim3 grid((max_k_len + 7) / 8, n);
    if (f32)
        latent_gather_kernel<float><<<grid, 256, 0, st>>>(static_cast<const float*>(kv), seqs, block_table, max_pages, n_pages, width, static_cast<float*>(out));
    else
        latent_gather_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(kv), seqs, block_table, max_pages, n_pages, width,
                                                                  static_cast<__nv_bfloat16*>(out));
    return cudaGetLastError();
}

bool latent_rows_has_kernel(int width, int rot_off) {
    return width % 16 == 0 && width <= 1024 && rot_off % 8 == 0 && rot_off <= 512 && rows_smem(width, 2) <= 220 * 1024;
}

cudaError_t launch_latent_rows(const LatentRowsParams& p, int rows, int n_splits, bool f32, bool plain, cudaStream_t st) {
    if (rows == 0) return cudaSuccess;
    if (rows > 65535) return cudaErrorInvalidValue;
    if (f32 || plain || !latent_rows_has_kernel(p.width, p.rot_off)) {
        const size_t smem = (size_t)(p.width + p.rot_off) * 4;
        if (smem > 220 * 1024) return cudaErrorInvalidValue;
        auto go = [&](auto kernel) {
            cudaError_t e = raise_smem(kernel, smem);
            return e != cudaSuccess ? e : launch_pdl(kernel, dim3(p.n_heads, rows), dim3(128), smem, st, p);
        };
        return f32 ? go(latent_plain_kernel<float>) : go(latent_plain_kernel<__nv_bfloat16>);
    }
    const int groups = (p.n_heads + 15) / 16;
    const dim3 grid(groups, n_splits, rows);
    auto go = [&](auto kernel, int stages) {
        const size_t smem = rows_smem(p.width, stages);
        cudaError_t e = raise_smem(kernel, smem);
        return e != cudaSuccess ? e : launch_pdl(kernel, grid, dim3(128), smem, st, p);
    };
    cudaError_t e;
    if (p.rot_off <= 64) e = go(latent_rows_kernel<2, 3>, 3);
    else if (p.rot_off <= 128) e = go(latent_rows_kernel<4, 3>, 3);
    else if (p.rot_off <= 256) e = go(latent_rows_kernel<8, 3>, 3);
    else e = go(latent_rows_kernel<16, 2>, 2);
    return e != cudaSuccess || n_splits == 1 ? e : launch_latent_merge(p, rows, n_splits, 16, st);
}

cudaError_t launch_latent_merge(const LatentRowsParams& p, int rows, int n_splits, int group, cudaStream_t st) {
    if (n_splits > MAX_SPLITS || rows > 65535) return cudaErrorInvalidValue;
    return launch_pdl(latent_merge_kernel, dim3(p.n_heads, rows), dim3(128), 0, st, p, n_splits, (p.n_heads + group - 1) / group, group);
}

bool latent_chunk_has_kernel(int dk, int dv) { return dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && dv <= 256; }

cudaError_t launch_latent_chunk(const LatentChunkParams& p, int n_seqs, int max_q_len, cudaStream_t st) {
    const int dk = p.dim + p.rot, dv = p.vdim;
    if (!latent_chunk_has_kernel(dk, dv) || p.dim % 8 || p.rot % 8 || p.n_heads > 65535 || n_seqs > 65535) return cudaErrorInvalidValue;
    const dim3 grid((max_q_len + BQ - 1) / BQ, p.n_heads, n_seqs);
    auto go = [&](auto kernel, size_t smem) {
        cudaError_t e = raise_smem(kernel, smem);
        if (e != cudaSuccess) return e;
        kernel<<<grid, 256, smem, st>>>(p);
        return cudaGetLastError();
    };
    if (dk <= 64 && dv <= 64) return go(latent_chunk_kernel<64, 64>, chunk_smem<64, 64>());
    if (dk <= 96 && dv <= 64) return go(latent_chunk_kernel<96, 64>, chunk_smem<96, 64>());
    if (dk <= 128 && dv <= 128) return go(latent_chunk_kernel<128, 128>, chunk_smem<128, 128>());
    if (dk <= 192 && dv <= 128) return go(latent_chunk_kernel<192, 128>, chunk_smem<192, 128>());
    return go(latent_chunk_kernel<256, 256>, chunk_smem<256, 256>());
}

LLM_DEFINE_BOUNDS_STATUS_READER(bounds_status_latent)

}  // namespace llm
