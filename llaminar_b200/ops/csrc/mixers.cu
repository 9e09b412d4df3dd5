// Mixers with a recurrent state: the row-wise kernels.
//
//   linear_rows    mLSTM and retention, row after row.  The state matrix S [vdim, dim] of a head is spread over a cluster of CTAs,
//                  which take slices of its rows: a warp reads whole rows of S, scales them, adds v k^T and multiplies by q while
//                  they pass through its registers, so the state is read and written once per token (what bounds a decode step).
//                  The CTAs of a cluster exchange the sums of squares of their slices through distributed shared memory for the
//                  norm of the head's output.
//   head_gate      norm and gate of the heads' outputs behind the chunk kernels (linear_tc.cu)
//   joint_gate     norm over all heads together and gate
#include <cooperative_groups.h>

#include "common.cuh"
#include "launch.h"
#include "mixers.h"

namespace llm {

namespace {

namespace cg = cooperative_groups;
constexpr float NORM_FLOOR = 1e-6f;            // of the mLSTM normaliser

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

LLM_DEVICE float sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

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

// ---- linear attention ------------------------------------------------------------------------------------------------------
constexpr int LIN_THREADS = 256, LIN_ROWS = 4;         // state rows in flight per warp

LLM_DEVICE float silu_exact(float x) { return x / (1.f + expf(-x)); }

// value i of a head's q or k: pairs (i, i + half) turn, the rest passes
template <class TI> LLM_DEVICE float rotated(const TI* x, int i, const float2* ang, int half) {
    if (i < half) return to_f(x[i]) * ang[i].x - to_f(x[i + half]) * ang[i].y;
    if (i < 2 * half) return to_f(x[i]) * ang[i - half].x + to_f(x[i - half]) * ang[i - half].y;
    return to_f(x[i]);
}

// Soft-capped log gates of one token and head: log input gate, log of the logistic forget gate
LLM_DEVICE void lstm_gates(float zi, float zf, float cap, float& i, float& f) {
    i = cap * tanhf(zi / cap);
    const float z = cap * tanhf(zf / cap);
    f = z >= 0.f ? -log1pf(expf(-z)) : z - log1pf(expf(z));
}

template <class TI, class TO>
__global__ void __launch_bounds__(LIN_THREADS, 3) linear_rows_kernel(const LinearParams p, int slice) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[LIN_THREADS / 32];
    __shared__ float s_sum[2][8];                      // the cluster's sums of squares, by token parity
    pdl_trigger();
    cg::cluster_group cluster = cg::this_cluster();
    const bool spread = gridDim.x > 1;                 // the head's rows are spread over the cluster
    if (spread) asm volatile("barrier.cluster.arrive.aligned;" ::: "memory");
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, D = p.dim;
    const int h = blockIdx.y, b = blockIdx.z, v0 = blockIdx.x * slice, nv = min(slice, p.vdim - v0);
    float *s_q = sm, *s_k = s_q + D, *s_n = s_k + D, *s_v = s_n + D, *s_o = s_v + slice;
    const int r0 = p.cu ? p.cu[b] : b, r1 = p.cu ? p.cu[b + 1] : b + 1;
    const int slot = LLM_CHECK_INDEX(p.slots[b], p.n_slots);
    const bool lstm = p.gates != nullptr;
    bool fresh = r0 < r1 && p.positions[r0] == 0;      // a sequence starts from zeros, whatever its slot holds
    float* S = p.S + (((size_t)slot * p.heads + h) * p.vdim + v0) * D;
    float* n_pool = lstm ? p.n + ((size_t)slot * p.heads + h) * D : nullptr;
    float* m_pool = lstm ? p.m + (size_t)slot * p.heads + h : nullptr;
    // a warp's first rows of the state are on their way before the rows in front of them are complete: slots, positions and the
    // sequences' rows come from the host, the state from an earlier step
    const bool one_pass = D <= 128;
    const int c_own = lane * 4;
    float nxt[LIN_ROWS][4];
    auto fetch = [&](int r) {
#pragma unroll
        for (int j = 0; j < LIN_ROWS; ++j) {
#pragma unroll
            for (int e = 0; e < 4; ++e) nxt[j][e] = 0.f;
            if (!fresh && r + j < nv && c_own < D) load4(S + (size_t)(r + j) * D + c_own, nxt[j]);
        }
    };
    if (one_pass) fetch(warp * LIN_ROWS);
    pdl_wait();
    if (spread) asm volatile("barrier.cluster.wait.aligned;" ::: "memory");       // every CTA of the cluster runs: its memory may be written
    float m = lstm && !fresh ? *m_pool : 0.f;
    if (lstm) for (int i = threadIdx.x; i < D; i += LIN_THREADS) s_n[i] = fresh ? 0.f : n_pool[i];
    const TI* in = static_cast<const TI*>(p.in);
    TO* out = static_cast<TO*>(p.out);
    for (int t = r0; t < r1; ++t) {
        if (one_pass && t > r0) fetch(warp * LIN_ROWS);
        const TI* row = in + (size_t)t * p.in_row;
        const TI *q = row + p.q_off + h * D, *k = row + p.k_off + h * D, *v = row + p.v_off + h * p.vdim + v0;
        const float2* ang = p.half ? p.angles + (size_t)t * p.half : nullptr;
        float keep, add = 1.f, den = 1.f;
        if (lstm) {
            float gi, gf;
            const float* z = p.gates + (size_t)t * p.gate_row;
            lstm_gates(z[h] + p.bias_i[h], z[p.heads + h] + p.bias_f[h], p.cap, gi, gf);
            const float top = fmaxf(gf + m, gi);
            keep = expf(gf + m - top);
            add = expf(gi - top);
            m = top;
        } else {
            keep = p.decay[h];
        }
        float nq = 0.f;
        for (int i = threadIdx.x; i < D; i += LIN_THREADS) {
            float a = rotated(q, i, ang, p.half), c = rotated(k, i, ang, p.half);
            if (p.silu_in) { a = silu_exact(a); c = silu_exact(c); }
            a *= p.q_scale; c *= p.k_scale;
            s_q[i] = a;
            s_k[i] = c;
            if (lstm) {
                const float x = keep * s_n[i] + add * c;
                s_n[i] = x;
                nq += x * a;
            }
        }
        for (int i = threadIdx.x; i < nv; i += LIN_THREADS) s_v[i] = p.silu_in ? silu_exact(to_f(v[i])) : to_f(v[i]);
        if (lstm) den = 1.f / (fmaxf(fabsf(block_sum<LIN_THREADS>(nq, red)), expf(-m)) + NORM_FLOOR);
        else __syncthreads();
        for (int r = warp * LIN_ROWS; r < nv; r += LIN_THREADS / 32 * LIN_ROWS) {
            float acc[LIN_ROWS] = {};
            for (int c = c_own; c < D; c += 128) {
                float s[LIN_ROWS][4], kk[4], qq[4];
                if (one_pass) {
#pragma unroll
                    for (int j = 0; j < LIN_ROWS; ++j)
#pragma unroll
                        for (int e = 0; e < 4; ++e) s[j][e] = nxt[j][e];
                    fetch(r + LIN_THREADS / 32 * LIN_ROWS);
                } else {
#pragma unroll
                    for (int j = 0; j < LIN_ROWS; ++j) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
                        if (!fresh && r + j < nv) load4(S + (size_t)(r + j) * D + c, s[j]);
                    }
                }
                load4(s_k + c, kk); load4(s_q + c, qq);
#pragma unroll
                for (int j = 0; j < LIN_ROWS; ++j) {
                    if (r + j >= nv) continue;
                    const float w = add * s_v[r + j];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        s[j][e] = keep * s[j][e] + w * kk[e];
                        acc[j] += s[j][e] * qq[e];
                    }
                    store4(S + (size_t)(r + j) * D + c, s[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < LIN_ROWS; ++j) {
                const float a = warp_sum(acc[j]);
                if (lane == 0 && r + j < nv) s_o[r + j] = a;
            }
        }
        __syncthreads();
        if (p.raw) {
            for (int i = threadIdx.x; i < nv; i += LIN_THREADS) out[(size_t)t * p.out_row + h * p.vdim + v0 + i] = from_f<TO>(s_o[i] * den);
            fresh = false;
            __syncthreads();
            continue;
        }
        float ss = 0.f;
        for (int i = threadIdx.x; i < nv; i += LIN_THREADS) { const float o = s_o[i] * den; ss += o * o; }
        ss = block_sum<LIN_THREADS>(ss, red);
        if (spread) {
            const int par = (t - r0) & 1;
            if (threadIdx.x < gridDim.x) *cluster.map_shared_rank(&s_sum[par][blockIdx.x], threadIdx.x) = ss;
            cluster.sync();
            ss = 0.f;
            for (int c = 0; c < (int)gridDim.x; ++c) ss += s_sum[par][c];
        }
        const float inv = den / sqrtf(ss / (float)p.true_vdim + p.eps);
        for (int i = threadIdx.x; i < nv; i += LIN_THREADS) {
            const int col = h * p.vdim + v0 + i;
            const float z = to_f(row[p.g_off + col]);
            float o = s_o[i] * inv * (p.silu ? z : 1.f) / (1.f + expf(-z));
            if (p.norm_w) o *= p.norm_w[col];
            out[(size_t)t * p.out_row + col] = from_f<TO>(o);
        }
        fresh = false;
        __syncthreads();                               // shared arrays are filled anew for the next token
    }
    if (spread) cluster.sync();                        // every CTA has read n and m
    if (lstm && blockIdx.x == 0 && r0 < r1) {
        for (int i = threadIdx.x; i < D; i += LIN_THREADS) n_pool[i] = s_n[i];
        if (threadIdx.x == 0) *m_pool = m;
    }
}

// a warp per token and head
__global__ void __launch_bounds__(256) head_gate_kernel(const LinearParams p, const __nv_bfloat16* o, int rows) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, unit = blockIdx.x * 8 + (threadIdx.x >> 5);
    const int t = unit / p.heads, h = unit - t * p.heads, col0 = h * p.vdim;
    if (t >= rows) return;
    const __nv_bfloat16* src = o + (size_t)t * p.heads * p.vdim + col0;
    const __nv_bfloat16* g = static_cast<const __nv_bfloat16*>(p.in) + (size_t)t * p.in_row + p.g_off + col0;
    __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + (size_t)t * p.out_row + col0;
    constexpr int UN = 2;                              // units of eight values a lane keeps; wider heads are read again
    uint4 keep[UN];
    float ss = 0.f;
    for (int i = 0; i * 256 < p.vdim; ++i) {
        const int c = i * 256 + lane * 8;
        const uint4 w = c < p.vdim ? *reinterpret_cast<const uint4*>(src + c) : make_uint4(0, 0, 0, 0);
        const uint32_t x[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) { const float a = bf16_lo(x[j]), b = bf16_hi(x[j]); ss += a * a + b * b; }
#pragma unroll
        for (int u = 0; u < UN; ++u) if (u == i) keep[u] = w;
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.true_vdim + p.eps);
    for (int i = 0; i * 256 < p.vdim; ++i) {
        const int c = i * 256 + lane * 8;
        if (c >= p.vdim) break;
        uint4 w = keep[0];
        if (i == 1) w = keep[1];
        if (i >= UN) w = *reinterpret_cast<const uint4*>(src + c);
        const uint4 z = *reinterpret_cast<const uint4*>(g + c);
        const uint32_t x[4] = {w.x, w.y, w.z, w.w}, y[4] = {z.x, z.y, z.z, z.w};
        uint32_t r[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float za = bf16_lo(y[j]), zb = bf16_hi(y[j]);
            float a = bf16_lo(x[j]) * inv * (p.silu ? za : 1.f) * sigmoid(za), b = bf16_hi(x[j]) * inv * (p.silu ? zb : 1.f) * sigmoid(zb);
            if (p.norm_w) { a *= p.norm_w[col0 + c + 2 * j]; b *= p.norm_w[col0 + c + 2 * j + 1]; }
            r[j] = pack_bf16(a, b);
        }
        *reinterpret_cast<uint4*>(dst + c) = make_uint4(r[0], r[1], r[2], r[3]);
    }
}

// a CTA per token
template <class TI, class T>
__global__ void __launch_bounds__(256, 5) joint_gate_kernel(const JointGateParams p) {
    __shared__ float red[8];
    pdl_trigger();
    pdl_wait();
    const size_t t = blockIdx.x;
    const TI *o = static_cast<const TI*>(p.o) + t * p.o_row, *g = static_cast<const TI*>(p.in) + t * p.in_row + p.g_off;
    T* dst = static_cast<T*>(p.out) + t * p.out_row;
    constexpr int UN = 2;                              // units of eight values a thread keeps; the rest of wider rows is read again
    auto load8 = [](const auto* s, float (&v)[8]) {
        float a[4], b[4];
        load4(s, a); load4(s + 4, b);
#pragma unroll
        for (int j = 0; j < 4; ++j) { v[j] = a[j]; v[4 + j] = b[j]; }
    };
    float keep[UN][8], z[UN][8], w[8], ss = 0.f;
#pragma unroll
    for (int u = 0; u < UN; ++u) {
        const int i = (u * 256 + threadIdx.x) * 8;
#pragma unroll
        for (int j = 0; j < 8; ++j) keep[u][j] = 0.f;
        if (i < p.n) { load8(o + i, keep[u]); load8(g + i, z[u]); }
    }
#pragma unroll
    for (int u = 0; u < UN; ++u)
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += keep[u][j] * keep[u][j];
    for (int i = (UN * 256 + threadIdx.x) * 8; i < p.n; i += 2048) {
        float x[8];
        load8(o + i, x);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
    }
    const float inv = 1.f / sqrtf(block_sum<256>(ss, red) / (float)p.true_n + p.eps);
    auto put = [&](int i, const float (&v)[8], const float (&s)[8]) {
        float a[4], b[4];
        load8(p.norm_w + i, w);
        auto value = [&](int j) {
            if constexpr (sizeof(T) == 2) return v[j] * inv * w[j] * sigmoid(s[j]);
            else return v[j] * inv * w[j] / (1.f + expf(-s[j]));
        };
#pragma unroll
        for (int j = 0; j < 4; ++j) { a[j] = value(j); b[j] = value(4 + j); }
        store4(dst + i, a); store4(dst + i + 4, b);
    };
#pragma unroll
    for (int u = 0; u < UN; ++u) {
        const int i = (u * 256 + threadIdx.x) * 8;
        if (i < p.n) put(i, keep[u], z[u]);
    }
    for (int i = (UN * 256 + threadIdx.x) * 8; i < p.n; i += 2048) {
        float x[8], s[8];
        load8(o + i, x); load8(g + i, s);
        put(i, x, s);
    }
}

}  // namespace

cudaError_t launch_joint_gate(const JointGateParams& p, int rows, bool in_f32, bool f32, cudaStream_t st) {
    if (rows == 0) return cudaSuccess;
    if (p.n % 8 || p.o_row % 8 || p.in_row % 8 || p.g_off % 8 || p.out_row % 8 || (f32 && !in_f32)) return cudaErrorInvalidValue;
    auto go = [&](auto kernel) { return launch_pdl(kernel, dim3(rows), dim3(256), 0, st, p); };
    if (f32) return go(joint_gate_kernel<float, float>);
    return in_f32 ? go(joint_gate_kernel<float, __nv_bfloat16>) : go(joint_gate_kernel<__nv_bfloat16, __nv_bfloat16>);
}

cudaError_t launch_linear_rows(const LinearParams& p, int n_seqs, bool in_f32, bool f32, cudaStream_t st) {
    if (n_seqs == 0) return cudaSuccess;
    if (p.dim % 8 || p.vdim % 8 || p.heads > 65535 || n_seqs > 65535 || (f32 && !in_f32) || (!p.gates == !p.decay)) return cudaErrorInvalidValue;
    // slices of at least 32 state rows: enough CTAs to fill the machine, clusters of at most eight
    int slices = 1;
    while (slices < 8 && p.vdim > 32 * slices && p.heads * n_seqs * slices < 2 * 148) slices *= 2;
    while ((p.vdim + slices - 1) / slices > 1024 && slices < 8) slices *= 2;
    const int slice = ((p.vdim + slices - 1) / slices + 7) / 8 * 8;
    slices = (p.vdim + slice - 1) / slice;
    const size_t smem = (size_t)(3 * p.dim + 2 * slice) * 4;
    if (smem > 48 * 1024) return cudaErrorInvalidValue;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(slices, p.heads, n_seqs);
    cfg.blockDim = dim3(LIN_THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = slices; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl_enabled() ? 2 : 1;
    if (f32) return cudaLaunchKernelEx(&cfg, linear_rows_kernel<float, float>, p, slice);
    return in_f32 ? cudaLaunchKernelEx(&cfg, linear_rows_kernel<float, __nv_bfloat16>, p, slice)
                  : cudaLaunchKernelEx(&cfg, linear_rows_kernel<__nv_bfloat16, __nv_bfloat16>, p, slice);
}

cudaError_t launch_head_gate(const LinearParams& p, const __nv_bfloat16* o, int rows, cudaStream_t st) {
    if (rows == 0) return cudaSuccess;
    if (p.vdim % 8 || p.in_row % 8 || p.g_off % 8 || p.out_row % 8) return cudaErrorInvalidValue;
    return launch_pdl(head_gate_kernel, dim3(((size_t)rows * p.heads + 7) / 8), dim3(256), 0, st, p, o, rows);
}

LLM_DEFINE_BOUNDS_STATUS_READER(bounds_status_mixers)

}  // namespace llm
