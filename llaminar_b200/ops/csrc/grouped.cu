// Around grouped-query attention: the row-wise kernels.
//
//   attn_prep      norms of the queries and keys over all heads together, append to the paged cache
//   head_prep      norms of queries and keys per head, rotation, append to the paged cache
//   conv_prep      short convolution over time, rotation, temperatures, mixing of values, append to the paged cache
//   conv_keep      the last rows of prompt portions into the convolution's state
//   attn_plain     one row and head per CTA in float arithmetic
#include "common.cuh"
#include "grouped.h"
#include "launch.h"

namespace llm {

namespace {

constexpr int PAGE = 64;

LLM_DEVICE float to_f(float v) { return v; }
LLM_DEVICE float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <class T> LLM_DEVICE T from_f(float v);
template <> LLM_DEVICE float from_f<float>(float v) { return v; }
template <> LLM_DEVICE __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

LLM_DEVICE void load4(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
LLM_DEVICE void load4(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    v[0] = bf16_lo(a.x); v[1] = bf16_hi(a.x); v[2] = bf16_lo(a.y); v[3] = bf16_hi(a.y);
}
LLM_DEVICE void store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
LLM_DEVICE void store4(__nv_bfloat16* p, const float (&v)[4]) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3])); }

template <int THREADS>
LLM_DEVICE float block_sum(float v, float* red) {
    v = warp_sum(v);
    __syncthreads();                               // red may still be read from the sum before
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; ++i) s += red[i];
    return s;
}

template <class TI, class T>
__global__ void __launch_bounds__(256) attn_prep_kernel(const AttnPrepParams p) {
    __shared__ float red[8];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const TI* row = static_cast<const TI*>(p.in) + (size_t)t * p.in_row;
    const TI *q = row + p.q_off, *k = row + p.k_off, *v = row + p.v_off;
    const int nq = p.n_heads * p.dim, nk = p.n_kv_heads * p.dim;
    const int pos = p.positions[t], seq = LLM_CHECK_INDEX(p.seq_ids[t], p.n_seqs);
    const int page = LLM_CHECK_INDEX(p.block_table[(size_t)seq * p.max_pages + pos / PAGE], p.n_pages);
    float sq = 0.f, sk = 0.f, x[4], w[4];
    for (int i = threadIdx.x * 4; i < nq; i += 1024) {
        load4(q + i, x);
#pragma unroll
        for (int j = 0; j < 4; ++j) sq += x[j] * x[j];
    }
    for (int i = threadIdx.x * 4; i < nk; i += 1024) {
        load4(k + i, x);
#pragma unroll
        for (int j = 0; j < 4; ++j) sk += x[j] * x[j];
    }
    const float iq = 1.f / sqrtf(block_sum<256>(sq, red) / (float)(p.n_heads * p.true_dim) + p.eps);
    const float ik = 1.f / sqrtf(block_sum<256>(sk, red) / (float)(p.n_kv_heads * p.true_dim) + p.eps);
    T* qo = static_cast<T*>(p.q_out) + (size_t)t * nq;
    for (int i = threadIdx.x * 4; i < nq; i += 1024) {
        load4(q + i, x); load4(p.q_norm + i, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] *= iq * w[j];
        store4(qo + i, x);
    }
    for (int i = threadIdx.x * 4; i < nk; i += 1024) {
        const int g = i / p.dim, c = i - g * p.dim;
        T* dst = static_cast<T*>(p.kv) + (((size_t)page * 2 * p.n_kv_heads + g) * PAGE + pos % PAGE) * p.dim + c;
        load4(k + i, x); load4(p.k_norm + i, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] *= ik * w[j];
        store4(dst, x);
        load4(v + i, x);
        store4(dst + (size_t)p.n_kv_heads * PAGE * p.dim, x);
    }
}

// The angles of values c .. c + 3 where all four lie on one side of the pairs (half % 4 == 0, c < 2 half)
struct Angles4 { float4 a, b; };
LLM_DEVICE Angles4 angles4(const float2* ang, int c, int half) {
    const int k = c < half ? c : c - half;
    return {*reinterpret_cast<const float4*>(ang + k), *reinterpret_cast<const float4*>(ang + k + 2)};
}
LLM_DEVICE void turned4(const float* row, int c, int half, const Angles4& g, float (&x)[4]) {
    const float co[4] = {g.a.x, g.a.z, g.b.x, g.b.z}, si[4] = {g.a.y, g.a.w, g.b.y, g.b.w};
    float y[4];
    load4(row + (c < half ? c + half : c - half), y);
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] = x[e] * co[e] + (c < half ? -y[e] : y[e]) * si[e];
}
// values c .. c + 3 of a row, rotated: pairs (i, i + half) turn, the rest passes
LLM_DEVICE void rotated4(const float* row, int c, int half, const float2* ang, float (&x)[4]) {
    load4(row + c, x);
    if (half % 4 == 0) {
        if (c < 2 * half) turned4(row, c, half, angles4(ang, c, half), x);
        return;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const int k = c + e;
        if (k < half) x[e] = x[e] * ang[k].x - row[k + half] * ang[k].y;
        else if (k < 2 * half) x[e] = x[e] * ang[k - half].x + row[k - half] * ang[k - half].y;
    }
}

// a warp per token and head: norm, rotation, and the append of keys and values
template <class TI, class T>
__global__ void __launch_bounds__(256) head_prep_kernel(const HeadPrepParams p) {
    extern __shared__ __align__(16) float sm[];                // [8][dim]
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x, D = p.dim, H = p.n_heads, G = p.n_kv_heads;
    const int u = blockIdx.y * 8 + warp;                       // queries, then keys, then values
    if (u >= H + 2 * G) return;
    const int kind = u < H ? 0 : u < H + G ? 1 : 2, h = u - (kind == 0 ? 0 : kind == 1 ? H : H + G);
    T* dst = static_cast<T*>(p.q_out) + ((size_t)t * H + h) * D;
    if (kind) {
        const int pos = p.positions[t], seq = LLM_CHECK_INDEX(p.seq_ids[t], p.n_seqs);
        const int page = LLM_CHECK_INDEX(p.block_table[(size_t)seq * p.max_pages + pos / PAGE], p.n_pages);
        dst = static_cast<T*>(p.kv) + ((((size_t)page * 2 + kind - 1) * G + h) * PAGE + pos % PAGE) * D;
    }
    pdl_wait();
    const TI* src = static_cast<const TI*>(p.in) + (size_t)t * p.in_row + (kind == 0 ? p.q_off : kind == 1 ? p.k_off : p.v_off) + (size_t)h * D;
    float x[4], w[4];
    if (kind == 2) {
        for (int i = lane * 4; i < D; i += 128) { load4(src + i, x); store4(dst + i, x); }
        return;
    }
    float* row = sm + warp * D;
    const float* gain = kind ? p.k_norm : p.q_norm;
    float ss = 0.f;
    for (int i = lane * 4; i < D; i += 128) {
        load4(src + i, x);
#pragma unroll
        for (int j = 0; j < 4; ++j) ss += x[j] * x[j];
        store4(row + i, x);
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.true_dim + p.eps);
    for (int i = lane * 4; i < D; i += 128) {                  // every lane reads back what it wrote
        load4(row + i, x); load4(gain + i, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] *= inv * w[j];
        store4(row + i, x);
    }
    __syncwarp();
    const float2* ang = p.angles + (size_t)t * p.half;
    for (int i = lane * 4; i < D; i += 128) {
        rotated4(row, i, p.half, ang, x);
        store4(dst + i, x);
    }
}

// A warp per head (queries, then keys, then values) and strip of N rows.  TAPS taps with at most four values per lane (dim <= 128): taps
// and the rows before the current one stay in registers, the next row and its angles are on their way; TAPS = 0: any number and size,
// N = 1.  Lane i looks up the strip's row i.
template <class TI, class T, int TAPS, int N>
__global__ void __launch_bounds__(256, N > 1 ? 3 : 4) conv_prep_kernel(const ConvPrepParams p) {
    extern __shared__ __align__(16) float sm[];                // [8][dim]
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, D = p.dim, H = p.n_heads, G = p.n_kv_heads, U = H + 2 * G;
    const int u = blockIdx.y * 8 + warp, t0 = blockIdx.x * N, t1 = min(t0 + N, p.rows), n_taps = TAPS ? TAPS : p.n_taps;
    if (u >= U) return;
    const int kind = u < H ? 0 : u < H + G ? 1 : 2, h = u - (kind == 0 ? 0 : kind == 1 ? H : H + G), col = u * D, cols = U * D;
    float* out = sm + warp * D;
    constexpr int KEEP = TAPS > 1 ? TAPS - 1 : 1;
    float w[TAPS ? TAPS : 1][4], past[KEEP][4], cur[4], nxt[4] = {};        // past[j]: the row j + 1 before the current one
    const int c_own = lane * 4;
    if constexpr (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            w[j][0] = w[j][1] = w[j][2] = w[j][3] = 0.f;
            if (c_own < D) load4(p.taps + (size_t)j * cols + col + c_own, w[j]);
        }
    }
    const TI* in = static_cast<const TI*>(p.in) + col;
    // positions and sequences come from the host
    int own_pos = 0, own_seq = 0, own_page = 0;
    if (lane < t1 - t0) {
        own_pos = p.positions[t0 + lane];
        own_seq = LLM_CHECK_INDEX(p.seq_ids[t0 + lane], p.n_seqs);
        if (kind) own_page = LLM_CHECK_INDEX(p.block_table[(size_t)own_seq * p.max_pages + own_pos / PAGE], p.n_pages);
    }
    int seq = __shfl_sync(0xffffffffu, own_seq, 0), r0 = p.cu ? p.cu[seq] : t0;          // r0: first row of the sequence's portion
    float* ring = p.ring + (size_t)LLM_CHECK_INDEX(p.slots[seq], p.n_slots) * n_taps * cols + col;
    const bool ahead = TAPS > 0 && kind < 2 && p.half % 4 == 0 && c_own < 2 * p.half;    // this lane's angles come as two vectors
    Angles4 ang_n = {};
    const float gain = kind == 0 && p.q_gain ? p.q_gain[h] : 1.f, share = p.share ? *p.share : 0.f;
    pdl_wait();
    if (TAPS > 0 && c_own < D) load4(in + (size_t)t0 * p.in_row + c_own, nxt);
    if (ahead) ang_n = angles4(p.angles + (size_t)t0 * p.half, c_own, p.half);
#pragma unroll 1
    for (int t = t0; t < t1; ++t) {
        const int pos = __shfl_sync(0xffffffffu, own_pos, t - t0), page = __shfl_sync(0xffffffffu, own_page, t - t0);
        const int seq_t = __shfl_sync(0xffffffffu, own_seq, t - t0);
        if (seq_t != seq) {                                    // the first row of another sequence's portion
            seq = seq_t;
            r0 = t;
            ring = p.ring + (size_t)LLM_CHECK_INDEX(p.slots[seq], p.n_slots) * n_taps * cols + col;
        }
        T* dst = static_cast<T*>(p.q_out) + ((size_t)t * H + h) * D;
        if (kind) dst = static_cast<T*>(p.kv) + ((((size_t)page * 2 + kind - 1) * G + h) * PAGE + pos % PAGE) * D;
        const Angles4 ang_t = ang_n;
        // what stood `lag` rows before this one, zeros in front of the sequence
        auto row_before = [&](int lag, int c, float (&x)[4]) {
            x[0] = x[1] = x[2] = x[3] = 0.f;
            if (c >= D || pos < lag) return;
            if (t - lag >= r0) load4(in + (size_t)(t - lag) * p.in_row + c, x);
            else load4(ring + (size_t)((pos - lag) % n_taps) * cols + c, x);
        };
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int e = 0; e < 4; ++e) cur[e] = nxt[e];
            if (t + 1 < t1 && c_own < D) load4(in + (size_t)(t + 1) * p.in_row + c_own, nxt);
            if (t + 1 < t1 && ahead) ang_n = angles4(p.angles + (size_t)(t + 1) * p.half, c_own, p.half);
            if (t == t0 || t == r0) {
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j) row_before(j + 1, c_own, past[j]);
            }
            if (c_own < D) {
                float a[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) a[e] = w[TAPS - 1][e] * cur[e];
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
                    for (int e = 0; e < 4; ++e) a[e] = fmaf(w[TAPS - 2 - j][e], past[j][e], a[e]);
                store4(out + c_own, a);
                if (!p.cu) store4(ring + (size_t)(pos % n_taps) * cols + c_own, cur);
            }
#pragma unroll
            for (int j = KEEP - 1; j >= 0; --j)
#pragma unroll
                for (int e = 0; e < 4; ++e) past[j][e] = j ? past[j - 1][e] : cur[e];
        } else {
            for (int c = c_own; c < D; c += 128) {
                float a[4] = {}, x[4], k[4];
                for (int lag = n_taps - 1; lag >= 0; --lag) {
                    if (lag) row_before(lag, c, x);
                    else load4(in + (size_t)t * p.in_row + c, x);
                    load4(p.taps + (size_t)(n_taps - 1 - lag) * cols + col + c, k);
#pragma unroll
                    for (int e = 0; e < 4; ++e) a[e] = fmaf(k[e], x[e], a[e]);
                }
                store4(out + c, a);
                if (!p.cu) store4(ring + (size_t)(pos % n_taps) * cols + c, x);
            }
        }
        float x[4];
        if (kind == 2) {
            float* first = p.first ? p.first + ((size_t)t * G + h) * p.first_dim : nullptr;
            for (int c = c_own; c < D; c += 128) {             // every lane reads back what it wrote
                load4(out + c, x);
                if (first && c < p.first_dim) {
                    if (p.share) {
                        float f[4];
                        load4(first + c, f);
#pragma unroll
                        for (int e = 0; e < 4; ++e) x[e] = (1.f - share) * x[e] + share * f[e];
                    } else {
                        store4(first + c, x);
                    }
                }
                store4(dst + c, x);
            }
        } else {
            __syncwarp();
            const float2* ang = p.angles + (size_t)t * p.half;
            for (int c = c_own; c < D; c += 128) {
                if (ahead) {
                    load4(out + c, x);
                    turned4(out, c, p.half, ang_t, x);
                } else {
                    rotated4(out, c, p.half, ang, x);
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) x[e] *= gain;
                store4(dst + c, x);
            }
            __syncwarp();                                      // the row has been read
        }
    }
}

template <class TI>
__global__ void __launch_bounds__(256) conv_keep_kernel(const ConvPrepParams p) {
    pdl_trigger();
    pdl_wait();
    const int cols = (p.n_heads + 2 * p.n_kv_heads) * p.dim, c = (blockIdx.x * 256 + threadIdx.x) * 4, seq = blockIdx.y;
    if (c >= cols) return;
    float* ring = p.ring + (size_t)LLM_CHECK_INDEX(p.slots[seq], p.n_slots) * p.n_taps * cols + c;
    for (int r = max(p.cu[seq], p.cu[seq + 1] - p.n_taps + 1); r < p.cu[seq + 1]; ++r) {
        float x[4];
        load4(static_cast<const TI*>(p.in) + (size_t)r * p.in_row + c, x);
        store4(ring + (size_t)(p.positions[r] % p.n_taps) * cols, x);
    }
}

template <class TG, class T>
__global__ void __launch_bounds__(128) attn_plain_kernel(const AttnPlainParams p) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_score[64];
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, t = blockIdx.y, D = p.dim, g = h / (p.n_heads / p.n_kv_heads);
    float *sq = sm, *so = sm + D;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int pos = p.positions[t];
    const int* btab = p.block_table + (size_t)LLM_CHECK_INDEX(p.seq_ids[t], p.n_seqs) * p.max_pages;
    const T* q = static_cast<const T*>(p.q) + ((size_t)t * p.n_heads + h) * D;
    for (int i = threadIdx.x; i < D; i += 128) { sq[i] = to_f(q[i]); so[i] = 0.f; }
    __syncthreads();
    auto key_row = [&](int key, int which) {
        const int page = LLM_CHECK_INDEX(btab[key / PAGE], p.n_pages);
        return static_cast<const T*>(p.kv) + ((((size_t)page * 2 + which) * p.n_kv_heads + g) * PAGE + key % PAGE) * D;
    };
    float m = p.sink ? p.sink[h] : -INFINITY, l = p.sink ? 1.f : 0.f;
    for (int k0 = first_key(pos, p.window, p.chunk); k0 <= pos; k0 += 64) {
        const int n = min(64, pos + 1 - k0);
        for (int j = warp; j < n; j += 4) {
            const T* row = key_row(k0 + j, 0);
            float s = 0.f;
            for (int i = lane; i < D; i += 32) s = fmaf(sq[i], to_f(row[i]), s);
            s = warp_sum(s);
            s *= p.scale;
            if (lane == 0) s_score[j] = p.softcap > 0.f ? p.softcap * tanhf(s / p.softcap) : s;
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
        for (int i = threadIdx.x; i < D; i += 128) {
            float a = so[i] * c;
            for (int j = 0; j < n; ++j) a = fmaf(s_score[j], to_f(key_row(k0 + j, 1)[i]), a);
            so[i] = a;
        }
        __syncthreads();
    }
    T* o = static_cast<T*>(p.out) + ((size_t)t * p.n_heads + h) * D;
    for (int i = threadIdx.x; i < D; i += 128) {
        float v = so[i] / l;
        if (p.gate) v *= 1.f / (1.f + expf(-to_f(static_cast<const TG*>(p.gate)[(size_t)t * p.gate_row + (p.gate_heads ? (size_t)h : (size_t)h * D + i)])));
        o[i] = from_f<T>(v);
    }
}

}  // namespace

cudaError_t launch_head_prep(const HeadPrepParams& p, int rows, bool in_f32, bool f32, cudaStream_t st) {
    if (rows == 0) return cudaSuccess;
    const size_t smem = (size_t)8 * p.dim * 4;
    if (p.dim % 8 || p.in_row % 4 || p.q_off % 4 || p.k_off % 4 || p.v_off % 4 || 2 * p.half > p.dim || smem > 48 * 1024 || (f32 && !in_f32)) return cudaErrorInvalidValue;
    const dim3 grid(rows, (p.n_heads + 2 * p.n_kv_heads + 7) / 8);
    auto go = [&](auto kernel) { return launch_pdl(kernel, grid, dim3(256), smem, st, p); };
    if (f32) return go(head_prep_kernel<float, float>);
    return in_f32 ? go(head_prep_kernel<float, __nv_bfloat16>) : go(head_prep_kernel<__nv_bfloat16, __nv_bfloat16>);
}

cudaError_t launch_conv_prep(const ConvPrepParams& p, bool in_f32, bool f32, cudaStream_t st) {
    if (p.rows == 0) return cudaSuccess;
    const size_t smem = (size_t)8 * p.dim * 4;
    if (p.dim % 8 || p.in_row % 4 || p.first_dim % 4 || p.first_dim > p.dim || 2 * p.half > p.dim || p.n_taps < 1 || smem > 48 * 1024 || (f32 && !in_f32)) return cudaErrorInvalidValue;
    constexpr int STRIP = 8;
    const int groups = (p.n_heads + 2 * p.n_kv_heads + 7) / 8;
    const bool strips = p.rows >= STRIP * 64 && !in_f32, few = p.dim <= 128 && !f32;
    auto go = [&](auto kernel, int n) { return launch_pdl(kernel, dim3((p.rows + n - 1) / n, groups), dim3(256), smem, st, p); };
    using B = __nv_bfloat16;
#define LLM_CONV_PREP(TAPS) if (few && p.n_taps == TAPS) return in_f32 ? go(conv_prep_kernel<float, B, TAPS, 1>, 1) : strips ? go(conv_prep_kernel<B, B, TAPS, STRIP>, STRIP) : go(conv_prep_kernel<B, B, TAPS, 1>, 1)
    LLM_CONV_PREP(2);
    LLM_CONV_PREP(3);
    LLM_CONV_PREP(4);
#undef LLM_CONV_PREP
    if (f32) return go(conv_prep_kernel<float, float, 0, 1>, 1);
    return in_f32 ? go(conv_prep_kernel<float, B, 0, 1>, 1) : go(conv_prep_kernel<B, B, 0, 1>, 1);
}

cudaError_t launch_conv_keep(const ConvPrepParams& p, bool in_f32, cudaStream_t st) {
    if (p.rows == 0 || p.n_taps == 1) return cudaSuccess;
    if (!p.cu || p.n_seqs > 65535 || p.dim % 4 || p.in_row % 4) return cudaErrorInvalidValue;
    const dim3 grid(((p.n_heads + 2 * p.n_kv_heads) * p.dim + 1023) / 1024, p.n_seqs);
    return in_f32 ? launch_pdl(conv_keep_kernel<float>, grid, dim3(256), 0, st, p) : launch_pdl(conv_keep_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, p);
}

cudaError_t launch_attn_prep(const AttnPrepParams& p, int rows, bool in_f32, bool f32, cudaStream_t st) {
    if (rows == 0) return cudaSuccess;
    if (p.dim % 8 || p.in_row % 4 || p.q_off % 4 || p.k_off % 4 || p.v_off % 4 || (f32 && !in_f32)) return cudaErrorInvalidValue;
    auto go = [&](auto kernel) { return launch_pdl(kernel, dim3(rows), dim3(256), 0, st, p); };
    if (f32) return go(attn_prep_kernel<float, float>);
    return in_f32 ? go(attn_prep_kernel<float, __nv_bfloat16>) : go(attn_prep_kernel<__nv_bfloat16, __nv_bfloat16>);
}

cudaError_t launch_attn_plain(const AttnPlainParams& p, int rows, bool gate_f32, bool f32, cudaStream_t st) {
    if (rows == 0) return cudaSuccess;
    const size_t smem = (size_t)p.dim * 8;
    if (rows > 65535 || smem > 48 * 1024 || p.n_heads % p.n_kv_heads) return cudaErrorInvalidValue;
    auto go = [&](auto kernel) { return launch_pdl(kernel, dim3(p.n_heads, rows), dim3(128), smem, st, p); };
    if (f32) return gate_f32 ? go(attn_plain_kernel<float, float>) : go(attn_plain_kernel<__nv_bfloat16, float>);
    return gate_f32 ? go(attn_plain_kernel<float, __nv_bfloat16>) : go(attn_plain_kernel<__nv_bfloat16, __nv_bfloat16>);
}

LLM_DEFINE_BOUNDS_STATUS_READER(bounds_status_grouped)

}  // namespace llm
