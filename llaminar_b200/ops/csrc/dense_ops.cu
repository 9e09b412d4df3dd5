// Fused norms of the residual stream, the gated activation, rotary angles and the small-batch matrix product of models whose
// matrices are stored as bf16 (or float, 32-bit mode).
#include "common.cuh"
#include "latent.h"
#include "launch.h"

namespace llm {

namespace {

LLM_DEVICE float to_f(float v) { return v; }
LLM_DEVICE float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <class T> LLM_DEVICE T from_f(float v);
template <> LLM_DEVICE float from_f<float>(float v) { return v; }
template <> LLM_DEVICE __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

LLM_DEVICE float gelu_tanh(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <int THREADS>
LLM_DEVICE float block_sum(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; ++i) s += red[i];
    __syncthreads();
    return s;
}

template <class T> struct Vec4 {};
template <> struct Vec4<float> {
    LLM_DEVICE static void load(const float* p, float (&v)[4]) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    }
    LLM_DEVICE static void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Vec4<__nv_bfloat16> {
    LLM_DEVICE static void load(const __nv_bfloat16* p, float (&v)[4]) {
        const uint2 a = *reinterpret_cast<const uint2*>(p);
        v[0] = bf16_lo(a.x); v[1] = bf16_hi(a.x); v[2] = bf16_lo(a.y); v[3] = bf16_hi(a.y);
    }
    LLM_DEVICE static void store(__nv_bfloat16* p, const float (&v)[4]) {
        *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
    }
};

// VEC 4 needs d and every row stride to be multiples of 4 elements; VEC 1 takes any size.
template <class T, int VEC, int THREADS>
__global__ void __launch_bounds__(THREADS) resid_norm_kernel(const ResidNormParams p) {
    extern __shared__ __align__(16) float row[];              // [d]
    __shared__ float red[THREADS / 32];
    pdl_trigger();
    pdl_wait();
    const size_t t = blockIdx.x;
    float* h = p.h + t * p.d;
    auto load_t = [](const T* s, float (&v)[VEC]) {
        if constexpr (VEC == 4) Vec4<T>::load(s, v); else v[0] = to_f(*s);
    };
    auto load_f = [](const float* s, float (&v)[VEC]) {
        if constexpr (VEC == 4) Vec4<float>::load(s, v); else v[0] = *s;
    };
    auto store_t = [](T* s, const float (&v)[VEC]) {
        if constexpr (VEC == 4) Vec4<T>::store(s, v); else *s = from_f<T>(v[0]);
    };
    auto store_f = [](float* s, const float (&v)[VEC]) {
        if constexpr (VEC == 4) Vec4<float>::store(s, v); else *s = v[0];
    };
    float inv_y = 0.f;
    const T* y = nullptr;
    if (p.y) {
        const size_t r = p.y_rows ? (size_t)LLM_CHECK_INDEX(p.y_rows[t], p.n_y_rows) : t;
        y = static_cast<const T*>(p.y) + r * p.y_stride;
        float ss = 0.f;
        for (int i = threadIdx.x * VEC; i < p.d; i += THREADS * VEC) {
            float v[VEC];
            load_t(y + i, v);
#pragma unroll
            for (int j = 0; j < VEC; ++j) ss += v[j] * v[j];
            store_f(row + i, v);
        }
        ss = block_sum<THREADS>(ss, red);
        inv_y = 1.f / sqrtf(ss / (float)p.d + p.eps);
    }
    float ss = 0.f;
    for (int i = threadIdx.x * VEC; i < p.d; i += THREADS * VEC) {
        float v[VEC];
        if (y) {
            float w[VEC];
            load_f(row + i, v);
            load_f(p.w_post + i, w);
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] = v[j] * inv_y * w[j];
            if (p.add) {
                float a[VEC];
                load_f(h + i, a);
#pragma unroll
                for (int j = 0; j < VEC; ++j) v[j] += a[j];
            }
            store_f(h + i, v);
        } else {
            load_f(h + i, v);
        }
        if (p.copy0) store_t(static_cast<T*>(p.copy0) + t * p.copy_stride + i, v);
        if (p.copy1) store_t(static_cast<T*>(p.copy1) + t * p.copy_stride + i, v);
        store_f(row + i, v);
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += v[j] * v[j];
    }
    if (!p.w_next) return;
    ss = block_sum<THREADS>(ss, red);
    const float inv = 1.f / sqrtf(ss / (float)p.d + p.eps);
    T* xn = static_cast<T*>(p.xn) + t * p.d;
    for (int i = threadIdx.x * VEC; i < p.d; i += THREADS * VEC) {
        float v[VEC], w[VEC];
        load_f(row + i, v);
        load_f(p.w_next + i, w);
#pragma unroll
        for (int j = 0; j < VEC; ++j) v[j] = v[j] * inv * w[j];
        store_t(xn + i, v);
    }
}

template <class T>
__global__ void __launch_bounds__(256) gelu_mul_kernel(const T* gu, T* act, int ff) {
    pdl_trigger();
    pdl_wait();
    const T* g = gu + (size_t)blockIdx.y * 2 * ff;
    T* a = act + (size_t)blockIdx.y * ff;
    if (ff % 4 == 0) {
        const int i = (blockIdx.x * 256 + threadIdx.x) * 4;
        if (i >= ff) return;
        float x[4], u[4];
        Vec4<T>::load(g + i, x);
        Vec4<T>::load(g + ff + i, u);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] = gelu_tanh(x[j]) * u[j];
        Vec4<T>::store(a + i, x);
    } else {
        for (int i = (blockIdx.x * 256 + threadIdx.x) * 4; i < min(ff, (int)(blockIdx.x * 256 + threadIdx.x + 1) * 4); ++i)
            a[i] = from_f<T>(gelu_tanh(to_f(g[i])) * to_f(g[ff + i]));
    }
}

__global__ void rope_angles_kernel(const int* positions, const double* freqs, double magnitude, float2* out, int rows, int half) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= rows * half) return;
    // the angle is reduced in double precision, so that positions far beyond 2^24 radians of float keep their fraction
    double turns = (double)positions[i / half] * freqs[i % half] * 0.15915494309189535;
    turns -= rint(turns);
    float s, c;
    sincosf((float)(turns * 6.283185307179586), &s, &c);
    out[i] = make_float2((float)magnitude * c, (float)magnitude * s);
}

// A group of LPR lanes computes one output column for all M rows; x is staged in shared memory once per CTA, which walks
// over the columns with stride gridDim.x.  GELU: two weight rows (gate and up) per output column.
template <int M, int LPR, bool GELU, class TO>
__global__ void __launch_bounds__(256) gemv_dense_kernel(const GemvDenseParams p) {
    extern __shared__ __align__(16) uint8_t smem_x[];
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    constexpr int RPW = 32 / LPR;                               // columns per warp
    const int sub = lane / LPR, l = lane % LPR;
    const __nv_bfloat16* W = p.w + (size_t)blockIdx.y * p.w_z;
    const int units = p.k / 8;
    pdl_wait();
    uint4* sx = reinterpret_cast<uint4*>(smem_x);               // [M][units]
    for (int i = threadIdx.x; i < M * units; i += 256)
        sx[i] = *reinterpret_cast<const uint4*>(p.x + (size_t)blockIdx.y * p.x_z + (i / units) * p.x_row + (size_t)(i % units) * 8);
    __syncthreads();
    constexpr int UN = 4;
    for (int n0 = (blockIdx.x * 8 + warp) * RPW; n0 < p.n; n0 += gridDim.x * 8 * RPW) {
        const int n = n0 + sub;
        const bool live = n < p.n;
        const __nv_bfloat16* wr = W + (size_t)(live ? n : p.n - 1) * p.ldw;
        const __nv_bfloat16* wr2 = GELU ? wr + (size_t)p.n * p.ldw : wr;
        float acc[M] = {}, acc2[M] = {};
        auto fma8 = [&](const uint4& w, int u, float (&a)[M]) {
            const uint32_t ws[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
            for (int m = 0; m < M; ++m) {
                const uint4 xv = sx[m * units + u];
                const uint32_t xs[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    a[m] = fmaf(bf16_lo(ws[j]), bf16_lo(xs[j]), a[m]);
                    a[m] = fmaf(bf16_hi(ws[j]), bf16_hi(xs[j]), a[m]);
                }
            }
        };
        int u = l;
        for (; u + (UN - 1) * LPR < units; u += UN * LPR) {
            uint4 w[UN], w2[GELU ? UN : 1];
#pragma unroll
            for (int i = 0; i < UN; ++i) {
                w[i] = ldg_nc_v4(wr + (size_t)(u + i * LPR) * 8);
                if constexpr (GELU) w2[i] = ldg_nc_v4(wr2 + (size_t)(u + i * LPR) * 8);
            }
#pragma unroll
            for (int i = 0; i < UN; ++i) {
                fma8(w[i], u + i * LPR, acc);
                if constexpr (GELU) fma8(w2[i], u + i * LPR, acc2);
            }
        }
        for (; u < units; u += LPR) {
            fma8(ldg_nc_v4(wr + (size_t)u * 8), u, acc);
            if constexpr (GELU) fma8(ldg_nc_v4(wr2 + (size_t)u * 8), u, acc2);
        }
#pragma unroll
        for (int m = 0; m < M; ++m) {
#pragma unroll
            for (int o = LPR / 2; o > 0; o >>= 1) {
                acc[m] += __shfl_xor_sync(0xffffffffu, acc[m], o);
                if constexpr (GELU) acc2[m] += __shfl_xor_sync(0xffffffffu, acc2[m], o);
            }
            float v = acc[m];
            // the two halves are rounded like the stored projection of the unfused form
            if constexpr (GELU) v = gelu_tanh(__bfloat162float(__float2bfloat16(v))) * __bfloat162float(__float2bfloat16(acc2[m]));
            if (live && l == 0) static_cast<TO*>(p.out)[(size_t)blockIdx.y * p.o_z + m * p.o_row + n] = from_f<TO>(v);
        }
    }
}

template <class K> cudaError_t raise_smem(K kernel, size_t bytes) {
    if (bytes <= 48 * 1024) return cudaSuccess;
    return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

template <class T>
cudaError_t resid_norm_any(const ResidNormParams& p, int rows, cudaStream_t st) {
    const size_t smem = (size_t)p.d * 4;
    if (smem > 220 * 1024) return cudaErrorInvalidValue;
    const bool vec = p.d % 4 == 0 && p.y_stride % 4 == 0 && p.copy_stride % 4 == 0;
    auto go = [&](auto kernel, int threads) {
        cudaError_t e = raise_smem(kernel, smem);
        return e != cudaSuccess ? e : launch_pdl(kernel, dim3(rows), dim3(threads), smem, st, p);
    };
    if (vec && p.d <= 1024) return go(resid_norm_kernel<T, 4, 128>, 128);
    if (vec) return go(resid_norm_kernel<T, 4, 512>, 512);
    return go(resid_norm_kernel<T, 1, 256>, 256);
}

template <int M, class TO>
cudaError_t gemv_m(const GemvDenseParams& p, cudaStream_t st) {
    const int units = p.k / 8;
    const size_t smem = (size_t)M * p.k * 2;
    auto go = [&](auto kernel, int lpr) {
        cudaError_t e = raise_smem(kernel, smem);
        if (e != cudaSuccess) return e;
        const int cols = 8 * (32 / lpr);
        int gx = (p.n + cols - 1) / cols;
        const int cap = 148 * 8;
        if (gx > cap) gx = cap;
        return launch_pdl(kernel, dim3(gx, p.z), dim3(256), smem, st, p);
    };
    if (p.gelu) {
        if constexpr (sizeof(TO) == 2) return go(gemv_dense_kernel<M, 32, true, TO>, 32);
        return cudaErrorInvalidValue;
    }
    if (units <= 8) return go(gemv_dense_kernel<M, 8, false, TO>, 8);
    if (units <= 24) return go(gemv_dense_kernel<M, 16, false, TO>, 16);
    return go(gemv_dense_kernel<M, 32, false, TO>, 32);
}

}  // namespace

cudaError_t launch_resid_norm(const ResidNormParams& p, int rows, bool f32, cudaStream_t st) {
    return f32 ? resid_norm_any<float>(p, rows, st) : resid_norm_any<__nv_bfloat16>(p, rows, st);
}

cudaError_t launch_gelu_mul(const void* gu, void* act, int rows, int ff, bool f32, cudaStream_t st) {
    const dim3 grid((ff + 1023) / 1024, rows);
    if (rows > 65535) return cudaErrorInvalidValue;
    if (f32) return launch_pdl(gelu_mul_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(gu), static_cast<float*>(act), ff);
    return launch_pdl(gelu_mul_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<const __nv_bfloat16*>(gu), static_cast<__nv_bfloat16*>(act), ff);
}

cudaError_t launch_rope_angles(const int* positions, const double* freqs, double magnitude, float2* out, int rows, int half, cudaStream_t st) {
    if (rows * half == 0) return cudaSuccess;
    rope_angles_kernel<<<(rows * half + 127) / 128, 128, 0, st>>>(positions, freqs, magnitude, out, rows, half);
    return cudaGetLastError();
}

cudaError_t launch_gemv_dense(const GemvDenseParams& p, cudaStream_t st) {
    if (p.m < 1 || p.m > 4 || p.k % 8 || p.ldw % 8 || p.w_z % 8 || p.x_row % 8 || p.x_z % 8 || (size_t)p.m * p.k * 2 > 200 * 1024)
        return cudaErrorInvalidValue;
    auto by_m = [&](auto tag) {
        using TO = decltype(tag);
        switch (p.m) {
            case 1: return gemv_m<1, TO>(p, st);
            case 2: return gemv_m<2, TO>(p, st);
            case 3: return gemv_m<3, TO>(p, st);
            default: return gemv_m<4, TO>(p, st);
        }
    };
    return p.out_f32 ? by_m(float()) : by_m(__nv_bfloat16());
}

LLM_DEFINE_BOUNDS_STATUS_READER(bounds_status_dense)

}  // namespace llm
