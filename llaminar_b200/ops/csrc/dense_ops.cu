// Fused norms of the residual stream, activations, rotary angles and the small-batch matrix product of models whose matrices are
// stored as bf16 (or float, 32-bit mode).
#include "common.cuh"
#include "dense.h"
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

LLM_DEVICE float logistic(float x) { return 1.f / (1.f + expf(-x)); }

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
    extern __shared__ __align__(16) float row[];              // [d], with y2 [2][d]
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
    // 1 / root mean square of the row, after its mean (returned in `mean`, 0 unless `center`) is taken off
    auto norm_of = [&](const float* r, float sum, float ss, bool center, float& mean) {
        mean = 0.f;
        if (center) {
            mean = block_sum<THREADS>(sum, red) / (float)p.d;
            ss = 0.f;
            for (int i = threadIdx.x * VEC; i < p.d; i += THREADS * VEC) {
                float v[VEC];
                load_f(r + i, v);
#pragma unroll
                for (int j = 0; j < VEC; ++j) ss += (v[j] - mean) * (v[j] - mean);
            }
        }
        return 1.f / sqrtf(block_sum<THREADS>(ss, red) / (float)p.d + p.eps);
    };
    float inv_y = 0.f, mean_y = 0.f;
    const T* y = nullptr;
    auto y_row = [&](size_t i) { return static_cast<const T*>(p.y) + (p.y_rows ? (size_t)LLM_CHECK_INDEX(p.y_rows[i], p.n_y_rows) : i) * p.y_stride; };
    if (p.y) {
        y = y_row(p.n_parts ? t * p.n_parts : t);
        const T* y2 = p.y2 ? static_cast<const T*>(p.y2) + t * p.y2_stride : nullptr;
        float ss = 0.f, ss2 = 0.f, sum = 0.f;
        for (int i = threadIdx.x * VEC; i < p.d; i += THREADS * VEC) {
            float v[VEC];
            load_t(y + i, v);
            if (p.n_parts) {
                float u[VEC];
#pragma unroll
                for (int j = 0; j < VEC; ++j) v[j] *= p.y_w[t * p.n_parts];
                for (int q = 1; q < p.n_parts; ++q) {
                    load_t(y_row(t * p.n_parts + q) + i, u);
#pragma unroll
                    for (int j = 0; j < VEC; ++j) v[j] = fmaf(u[j], p.y_w[t * p.n_parts + q], v[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < VEC; ++j) { ss += v[j] * v[j]; sum += v[j]; }
            store_f(row + i, v);
            if (y2) {
                load_t(y2 + i, v);
#pragma unroll
                for (int j = 0; j < VEC; ++j) ss2 += v[j] * v[j];
                store_f(row + p.d + i, v);
            }
        }
        if (y2) {
            const float a = 0.5f / sqrtf(block_sum<THREADS>(ss, red) / (float)p.d + p.eps), b = 0.5f / sqrtf(block_sum<THREADS>(ss2, red) / (float)p.d + p.eps);
            ss = sum = 0.f;
            for (int i = threadIdx.x * VEC; i < p.d; i += THREADS * VEC) {      // every thread reads back what it wrote
                float v[VEC], u[VEC], w[VEC], x[VEC];
                load_f(row + i, v); load_f(row + p.d + i, u); load_f(p.w_y + i, w); load_f(p.w_y2 + i, x);
#pragma unroll
                for (int j = 0; j < VEC; ++j) { v[j] = v[j] * a * w[j] + u[j] * b * x[j]; ss += v[j] * v[j]; sum += v[j]; }
                store_f(row + i, v);
            }
        }
        inv_y = p.w_post ? norm_of(row, sum, ss, p.center_post, mean_y) : p.factor;
    }
    float ss = 0.f, sum = 0.f;
    for (int i = threadIdx.x * VEC; i < p.d; i += THREADS * VEC) {
        float v[VEC];
        if (y) {
            float w[VEC];
            load_f(row + i, v);
#pragma unroll
            for (int j = 0; j < VEC; ++j) w[j] = 1.f;
            if (p.w_post) load_f(p.w_post + i, w);
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] = (v[j] - mean_y) * inv_y * w[j];
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
        for (int j = 0; j < VEC; ++j) { ss += v[j] * v[j]; sum += v[j]; }
    }
    if (!p.w_next) return;
    float mean;
    const float inv = norm_of(row, sum, ss, p.center_next, mean);
    T* xn = static_cast<T*>(p.xn) + t * p.d;
    for (int i = threadIdx.x * VEC; i < p.d; i += THREADS * VEC) {
        float v[VEC], w[VEC];
        load_f(row + i, v);
        load_f(p.w_next + i, w);
#pragma unroll
        for (int j = 0; j < VEC; ++j) v[j] = (v[j] - mean) * inv * w[j];
        store_t(xn + i, v);
    }
}

// The same for rows that the threads hold in registers (NV x 4 values each): every load is on its way before the first sum.
template <class T, int THREADS, int NV, bool PARTS>                         // PARTS: y is a weighted sum of rows
__global__ void __launch_bounds__(THREADS) resid_norm_reg_kernel(const ResidNormParams p) {
    constexpr int W = THREADS / 32;
    __shared__ float2 red[5][W];
    pdl_trigger();
    const size_t t = blockIdx.x;
    const int d = p.d;
    float* h = p.h + t * d;
    auto at = [&](int n) { return (n * THREADS + (int)threadIdx.x) * 4; };
    auto each = [&](auto f) {
#pragma unroll
        for (int n = 0; n < NV; ++n)
            if (at(n) < d) f(n, at(n));
    };
    int used = 0;                                              // sums so far: each has its own place in `red`
    auto block_sum2 = [&](float x, float y) {
        x = warp_sum(x); y = warp_sum(y);
        float2(&r)[W] = red[used++];
        if ((threadIdx.x & 31) == 0) r[threadIdx.x >> 5] = make_float2(x, y);
        __syncthreads();
        float2 s = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < W; ++i) { s.x += r[i].x; s.y += r[i].y; }
        return s;
    };
    float v[NV][4], a[NV][4] = {}, w[NV][4];
    // mean (0 unless `center`) and 1 / root mean square around it
    auto norm_of = [&](bool center, float& mean) {
        float sum = 0.f, ss = 0.f;
        each([&](int n, int) {
#pragma unroll
            for (int j = 0; j < 4; ++j) { sum += v[n][j]; ss += v[n][j] * v[n][j]; }
        });
        const float2 s = block_sum2(sum, ss);
        mean = 0.f;
        ss = s.y;
        if (center) {
            mean = s.x / (float)d;
            float q = 0.f;
            each([&](int n, int) {
#pragma unroll
                for (int j = 0; j < 4; ++j) q += (v[n][j] - mean) * (v[n][j] - mean);
            });
            ss = block_sum2(q, 0.f).x;
        }
        return 1.f / sqrtf(ss / (float)d + p.eps);
    };
    if (p.y && p.w_post) each([&](int n, int i) { Vec4<float>::load(p.w_post + i, w[n]); });
    pdl_wait();
    if (!p.y || p.add) each([&](int n, int i) { Vec4<float>::load(h + i, a[n]); });
    if (p.y) {
        auto y_row = [&](size_t i) { return static_cast<const T*>(p.y) + (p.y_rows ? (size_t)LLM_CHECK_INDEX(p.y_rows[i], p.n_y_rows) : i) * p.y_stride; };
        if constexpr (PARTS) {
            each([&](int n, int) { v[n][0] = v[n][1] = v[n][2] = v[n][3] = 0.f; });
#pragma unroll 4
            for (int q = 0; q < p.n_parts; ++q) {
                const T* y = y_row(t * p.n_parts + q);
                const float w = p.y_w[t * p.n_parts + q];
                each([&](int n, int i) {
                    float u[4];
                    Vec4<T>::load(y + i, u);
#pragma unroll
                    for (int j = 0; j < 4; ++j) v[n][j] = fmaf(u[j], w, v[n][j]);
                });
            }
        } else {
            const T* y = y_row(t);
            each([&](int n, int i) { Vec4<T>::load(y + i, v[n]); });
        }
        if (p.y2) {
            const T* y2 = static_cast<const T*>(p.y2) + t * p.y2_stride;
            float u[NV][4], sa = 0.f, sb = 0.f;
            each([&](int n, int i) {
                Vec4<T>::load(y2 + i, u[n]);
#pragma unroll
                for (int j = 0; j < 4; ++j) { sa += v[n][j] * v[n][j]; sb += u[n][j] * u[n][j]; }
            });
            const float2 s = block_sum2(sa, sb);
            const float ia = 0.5f / sqrtf(s.x / (float)d + p.eps), ib = 0.5f / sqrtf(s.y / (float)d + p.eps);
            each([&](int n, int i) {
                float wa[4], wb[4];
                Vec4<float>::load(p.w_y + i, wa); Vec4<float>::load(p.w_y2 + i, wb);
#pragma unroll
                for (int j = 0; j < 4; ++j) v[n][j] = v[n][j] * ia * wa[j] + u[n][j] * ib * wb[j];
            });
        }
        float mean = 0.f;
        const float inv = p.w_post ? norm_of(p.center_post, mean) : p.factor;
        each([&](int n, int i) {
#pragma unroll
            for (int j = 0; j < 4; ++j) v[n][j] = a[n][j] + (v[n][j] - mean) * inv * (p.w_post ? w[n][j] : 1.f);
            Vec4<float>::store(h + i, v[n]);
        });
    } else {
        each([&](int n, int) {
#pragma unroll
            for (int j = 0; j < 4; ++j) v[n][j] = a[n][j];
        });
    }
    each([&](int n, int i) {
        if (p.copy0) Vec4<T>::store(static_cast<T*>(p.copy0) + t * p.copy_stride + i, v[n]);
        if (p.copy1) Vec4<T>::store(static_cast<T*>(p.copy1) + t * p.copy_stride + i, v[n]);
    });
    if (!p.w_next) return;
    float mean;
    const float inv = norm_of(p.center_next, mean);
    T* xn = static_cast<T*>(p.xn) + t * d;
    each([&](int n, int i) {
        Vec4<float>::load(p.w_next + i, w[n]);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[n][j] = (v[n][j] - mean) * inv * w[n][j];
        Vec4<T>::store(xn + i, v[n]);
    });
}

LLM_DEVICE void load8(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
LLM_DEVICE void load8(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 a = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) { v[2 * j] = bf16_lo(w[j]); v[2 * j + 1] = bf16_hi(w[j]); }
}
LLM_DEVICE void store8(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
LLM_DEVICE void store8(__nv_bfloat16* p, const float (&v)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}

// See DepthMixParams.  A CTA per row; a thread holds NV x VEC of its values (VEC = 1: of any alignment).
template <class T, int VEC, int THREADS, int NV, bool PARTS>
__global__ void __launch_bounds__(THREADS) depth_mix_kernel(const DepthMixParams p) {
    constexpr int W = THREADS / 32;
    __shared__ float red[W];
    pdl_trigger();
    const size_t t = blockIdx.x;
    const int d = p.d;
    auto at = [&](int n) { return (n * THREADS + (int)threadIdx.x) * VEC; };
    auto each = [&](auto f) {
#pragma unroll
        for (int n = 0; n < NV; ++n)
            if (at(n) < d) f(n, at(n));
    };
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
    pdl_wait();
    float* h = p.h + t * d;
    float v[NV][VEC] = {};
    const bool update = p.y || p.z;
    if (p.add || !update) each([&](int n, int i) { load_f(h + i, v[n]); });
    if (p.y) {
        const T* y = static_cast<const T*>(p.y) + (p.y_rows ? (size_t)LLM_CHECK_INDEX(p.y_rows[t], p.n_y_rows) : t) * p.y_stride;
        float u[NV][VEC];
        each([&](int n, int i) { load_t(y + i, u[n]); });
        each([&](int n, int) {
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[n][j] += u[n][j];
        });
    }
    if (p.z) {
        auto z_row = [&](size_t i) { return static_cast<const T*>(p.z) + (p.z_rows ? (size_t)LLM_CHECK_INDEX(p.z_rows[i], p.n_z_rows) : i) * p.z_stride; };
        if constexpr (PARTS) {
            float s[NV][VEC] = {};
#pragma unroll 4
            for (int q = 0; q < p.n_parts; ++q) {
                const T* z = z_row(t * p.n_parts + q);
                const float w = p.z_w[t * p.n_parts + q];
                each([&](int n, int i) {
                    float u[VEC];
                    load_t(z + i, u);
#pragma unroll
                    for (int j = 0; j < VEC; ++j) s[n][j] = fmaf(u[j], w, s[n][j]);
                });
            }
            each([&](int n, int) {
#pragma unroll
                for (int j = 0; j < VEC; ++j) v[n][j] += s[n][j];
            });
        } else {
            const T* z = z_row(t);
            each([&](int n, int i) {
                float u[VEC];
                load_t(z + i, u);
#pragma unroll
                for (int j = 0; j < VEC; ++j) v[n][j] += u[j];
            });
        }
    }
    if (p.keep) each([&](int n, int i) { store_f(p.past + p.n_past * p.past_stride + t * d + i, v[n]); });
    if (p.w) {
        const float own = p.w[p.n_past];
        each([&](int n, int) {
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[n][j] *= own;
        });
#pragma unroll 4
        for (int q = 0; q < p.n_past; ++q) {
            const float w = p.w[q];
            const float* x = p.past + q * p.past_stride + t * d;
            each([&](int n, int i) {
                float u[VEC];
                load_f(x + i, u);
#pragma unroll
                for (int j = 0; j < VEC; ++j) v[n][j] = fmaf(u[j], w, v[n][j]);
            });
        }
    }
    if (update) each([&](int n, int i) { store_f(h + i, v[n]); });
    if (!p.xn0 && !p.xn1) return;
    float ss = 0.f;
    each([&](int n, int) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += v[n][j] * v[n][j];
    });
    const float inv = 1.f / sqrtf(block_sum<THREADS>(ss, red) / (float)d + p.eps);
    auto norm = [&](const float* gain, void* xn) {
        if (!xn) return;
        each([&](int n, int i) {
            float u[VEC];
#pragma unroll
            for (int j = 0; j < VEC; ++j) u[j] = v[n][j] * inv * gain[(i + j) * p.gain_step];
            store_t(static_cast<T*>(xn) + t * d + i, u);
        });
    };
    norm(p.gain0, p.xn0);
    norm(p.gain1, p.xn1);
}

// For results that are rounded to 16 bits: approximate exponential and quotient (relative errors of some 1e-6).  gelu's
// (1 + tanh(w)) / 2 is the logistic function of 2w.
template <class T> LLM_DEVICE float logistic_for(float x) {
    if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-x));
    else return logistic(x);
}
template <class T> LLM_DEVICE float gelu_for(float z) {
    if constexpr (sizeof(T) == 2) return z * logistic_for<T>(1.5957691216057308f * (z + 0.044715f * z * z * z));
    else return gelu_tanh(z);
}

// value `i` of row `t` of the activation of `x`; `u`: the second half's value (GELU_MUL, SILU_MUL)
template <int ACT, class T>
LLM_DEVICE float activated(float x, float u, const SideTable& s, int t, int i) {
    if (ACT == ACT_GELU_MUL) return gelu_for<T>(x) * u;
    if (ACT == ACT_SILU_MUL) return x * logistic_for<T>(x) * u;
    if (ACT == ACT_GATE) return x * logistic_for<T>(to_f(static_cast<const T*>(s.table)[(size_t)t * s.row + i]));
    if (ACT == ACT_RELU2) { x = fmaxf(x, 0.f); return x * x; }
    if (ACT == ACT_GELU) return gelu_for<T>(x);
    if (ACT == ACT_SILU) return x * logistic_for<T>(x);
    if (ACT == ACT_GELU_SIDE) return i < s.cols ? gelu_for<T>(x) * to_f(static_cast<const T*>(s.table)[(size_t)LLM_CHECK_INDEX(s.tokens[t], s.n_rows) * s.row + i]) : 0.f;
    return x;
}

template <class T, int ACT>
__global__ void __launch_bounds__(256) activate_kernel(const T* x, size_t x_row, T* act, size_t act_row, int n, const SideTable s) {
    pdl_trigger();
    pdl_wait();
    const T* g = x + (size_t)blockIdx.y * x_row;
    T* a = act + (size_t)blockIdx.y * act_row;
    const int i0 = (blockIdx.x * 256 + threadIdx.x) * 8;
    if ((n | x_row | act_row) % 8 == 0) {
        if (i0 >= n) return;
        float v[8], u[8] = {};
        load8(g + i0, v);
        if (act_pairs(ACT)) load8(g + n + i0, u);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = activated<ACT, T>(v[j], u[j], s, blockIdx.y, i0 + j);
        store8(a + i0, v);
    } else {
        for (int i = i0; i < min(n, i0 + 8); ++i)
            a[i] = from_f<T>(activated<ACT, T>(to_f(g[i]), act_pairs(ACT) ? to_f(g[n + i]) : 0.f, s, blockIdx.y, i));
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

// Up to eight rows of x against 16 weight rows per warp on the tensor cores (the weights are the M operand).  Thread (g, t) of
// a warp loads 8 consecutive k of weight rows g and g + 8 and of x row g in one 16-byte access each; since both operands use
// the same assignment of k to MMA slots, its order does not matter and no operand passes through shared memory.  `wk` warps
// share the K range of a row block and add up in shared memory.  GELU_MUL, SILU_MUL: a second set of weight rows (n further down) per block.
constexpr int SKINNY_WARPS = 8;
LLM_DEVICE void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
template <int ACT, class TO>
__global__ void __launch_bounds__(32 * SKINNY_WARPS) gemv_dense_kernel(const GemvDenseParams p, int wk) {
    constexpr bool PAIR = act_pairs(ACT);
    __shared__ float s_acc[SKINNY_WARPS][PAIR ? 2 : 1][16][9];
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int part = warp % wk, n0 = (blockIdx.x * (SKINNY_WARPS / wk) + warp / wk) * 16;
    const int blocks = (p.k + 31) / 32, per = (blocks + wk - 1) / wk, kb0 = part * per, kb1 = min(blocks, kb0 + per);
    constexpr int UN = PAIR ? 4 : 8, NW = PAIR ? 4 : 2;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float acc[PAIR ? 2 : 1][4] = {};
    // rows past the end repeat the last one (never stored)
    const __nv_bfloat16* w[NW];
#pragma unroll
    for (int i = 0; i < NW; ++i) w[i] = p.w + (size_t)blockIdx.y * p.w_z + (size_t)(min(n0 + g + (i & 1) * 8, p.n - 1) + (i >> 1) * p.n) * p.ldw + t * 8;
    const __nv_bfloat16* x = p.x + (size_t)blockIdx.y * p.x_z + (size_t)min(g, p.m - 1) * p.x_row + t * 8;
    const bool live = n0 < p.n;
    bool waited = false;
    for (int kb = kb0; kb < kb1 && live; kb += UN) {
        uint4 wv[UN][NW], xv[UN];
#pragma unroll
        for (int u = 0; u < UN; ++u) {
            const bool in = kb + u < kb1 && (kb + u) * 32 + t * 8 < p.k;
#pragma unroll
            for (int i = 0; i < NW; ++i) wv[u][i] = in ? ldg_nc_v4(w[i] + (size_t)(kb + u) * 32) : zero;
        }
        if (!waited) { pdl_wait(); waited = true; }             // the first weights are on their way before x is complete
#pragma unroll
        for (int u = 0; u < UN; ++u) {
            const bool in = kb + u < kb1 && (kb + u) * 32 + t * 8 < p.k && g < p.m;
            xv[u] = in ? *reinterpret_cast<const uint4*>(x + (size_t)(kb + u) * 32) : zero;
        }
#pragma unroll
        for (int u = 0; u < UN; ++u) {
#pragma unroll
            for (int i = 0; i < NW / 2; ++i) {
                mma_bf16(acc[i], wv[u][2 * i].x, wv[u][2 * i + 1].x, wv[u][2 * i].y, wv[u][2 * i + 1].y, xv[u].x, xv[u].y);
                mma_bf16(acc[i], wv[u][2 * i].z, wv[u][2 * i + 1].z, wv[u][2 * i].w, wv[u][2 * i + 1].w, xv[u].z, xv[u].w);
            }
        }
    }
    if (!waited) pdl_wait();
#pragma unroll
    for (int i = 0; i < NW / 2; ++i) {
        s_acc[warp][i][g][2 * t] = acc[i][0]; s_acc[warp][i][g][2 * t + 1] = acc[i][1];
        s_acc[warp][i][g + 8][2 * t] = acc[i][2]; s_acc[warp][i][g + 8][2 * t + 1] = acc[i][3];
    }
    __syncthreads();
    // 16 columns x m rows per row block of the CTA
    const int rb = SKINNY_WARPS / wk;
    for (int i = threadIdx.x; i < rb * 16 * p.m; i += 32 * SKINNY_WARPS) {
        const int c = i % (rb * 16), m = i / (rb * 16), n = blockIdx.x * rb * 16 + c;
        if (n >= p.n) continue;
        float v = 0.f, v2 = 0.f;
        for (int q = 0; q < wk; ++q) {
            v += s_acc[(c / 16) * wk + q][0][c % 16][m];
            if constexpr (PAIR) v2 += s_acc[(c / 16) * wk + q][1][c % 16][m];
        }
        // rounded like the stored projection of the unfused form
        if constexpr (ACT != ACT_NONE)
            v = activated<ACT, __nv_bfloat16>(__bfloat162float(__float2bfloat16(v)), __bfloat162float(__float2bfloat16(v2)), p.side,
                                              ACT == ACT_GATE ? m : blockIdx.y * p.m + m, ACT == ACT_GATE ? blockIdx.y * p.n + n : n);
        static_cast<TO*>(p.out)[(size_t)blockIdx.y * p.o_z + m * p.o_row + n] = from_f<TO>(v);
    }
}

template <class K> cudaError_t raise_smem(K kernel, size_t bytes) {
    if (bytes <= 48 * 1024) return cudaSuccess;
    return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

template <class T>
cudaError_t resid_norm_any(const ResidNormParams& p, int rows, cudaStream_t st) {
    const size_t smem = (size_t)p.d * (p.y2 ? 8 : 4);
    if (smem > 220 * 1024) return cudaErrorInvalidValue;
    const bool vec = p.d % 4 == 0 && p.y_stride % 4 == 0 && p.y2_stride % 4 == 0 && p.copy_stride % 4 == 0;
    auto go = [&](auto kernel, int threads) {
        cudaError_t e = raise_smem(kernel, smem);
        return e != cudaSuccess ? e : launch_pdl(kernel, dim3(rows), dim3(threads), smem, st, p);
    };
    auto go_reg = [&](auto kernel, int threads) { return launch_pdl(kernel, dim3(rows), dim3(threads), 0, st, p); };
    if (vec && p.d <= 1024) return go_reg(p.n_parts ? resid_norm_reg_kernel<T, 128, 2, true> : resid_norm_reg_kernel<T, 128, 2, false>, 128);
    if (vec && p.d <= 2048) return go_reg(p.n_parts ? resid_norm_reg_kernel<T, 256, 2, true> : resid_norm_reg_kernel<T, 256, 2, false>, 256);
    if (vec && p.d <= 4096) return go_reg(p.n_parts ? resid_norm_reg_kernel<T, 512, 2, true> : resid_norm_reg_kernel<T, 512, 2, false>, 512);
    if (vec && p.d <= 8192) return go_reg(p.n_parts ? resid_norm_reg_kernel<T, 512, 4, true> : resid_norm_reg_kernel<T, 512, 4, false>, 512);
    if (vec) return go(resid_norm_kernel<T, 4, 512>, 512);
    return go(resid_norm_kernel<T, 1, 256>, 256);
}

}  // namespace

cudaError_t launch_depth_mix(const DepthMixParams& p, int rows, bool f32, cudaStream_t st) {
    if (rows == 0) return cudaSuccess;
    const bool vec = p.d % 4 == 0 && p.y_stride % 4 == 0 && p.z_stride % 4 == 0 && p.past_stride % 4 == 0;
    if (p.d < 1 || p.d > (vec ? 16384 : 8192) || (p.w == nullptr && p.n_past > 0)) return cudaErrorInvalidValue;
    auto go = [&](auto plain, auto parts, int threads) { return launch_pdl(p.n_parts ? parts : plain, dim3(rows), dim3(threads), 0, st, p); };
#define LLM_DEPTH_MIX(T, VEC, THREADS, NV) return go(depth_mix_kernel<T, VEC, THREADS, NV, false>, depth_mix_kernel<T, VEC, THREADS, NV, true>, THREADS)
    auto any = [&](auto tag) {
        using T = decltype(tag);
        if (!vec) LLM_DEPTH_MIX(T, 1, 512, 16);
        if (p.d <= 1024) LLM_DEPTH_MIX(T, 4, 128, 2);
        if (p.d <= 2048) LLM_DEPTH_MIX(T, 4, 256, 2);
        if (p.d <= 4096) LLM_DEPTH_MIX(T, 4, 512, 2);
        if (p.d <= 8192) LLM_DEPTH_MIX(T, 4, 512, 4);
        LLM_DEPTH_MIX(T, 4, 512, 8);
    };
#undef LLM_DEPTH_MIX
    return f32 ? any(float()) : any(__nv_bfloat16());
}

cudaError_t launch_resid_norm(const ResidNormParams& p, int rows, bool f32, cudaStream_t st) {
    return f32 ? resid_norm_any<float>(p, rows, st) : resid_norm_any<__nv_bfloat16>(p, rows, st);
}

cudaError_t launch_activate(const void* x, size_t x_row, void* act, size_t act_row, int rows, int n, int kind, const SideTable& side, bool f32, cudaStream_t st) {
    const dim3 grid((n + 2047) / 2048, rows);
    if (rows > 65535) return cudaErrorInvalidValue;
    auto go = [&](auto k32, auto k16) {
        if (f32) return launch_pdl(k32, grid, dim3(256), 0, st, static_cast<const float*>(x), x_row, static_cast<float*>(act), act_row, n, side);
        return launch_pdl(k16, grid, dim3(256), 0, st, static_cast<const __nv_bfloat16*>(x), x_row, static_cast<__nv_bfloat16*>(act), act_row, n, side);
    };
    if (kind == ACT_GELU_MUL) return go(activate_kernel<float, ACT_GELU_MUL>, activate_kernel<__nv_bfloat16, ACT_GELU_MUL>);
    if (kind == ACT_SILU_MUL) return go(activate_kernel<float, ACT_SILU_MUL>, activate_kernel<__nv_bfloat16, ACT_SILU_MUL>);
    if (kind == ACT_GATE) return go(activate_kernel<float, ACT_GATE>, activate_kernel<__nv_bfloat16, ACT_GATE>);
    if (kind == ACT_RELU2) return go(activate_kernel<float, ACT_RELU2>, activate_kernel<__nv_bfloat16, ACT_RELU2>);
    if (kind == ACT_GELU) return go(activate_kernel<float, ACT_GELU>, activate_kernel<__nv_bfloat16, ACT_GELU>);
    if (kind == ACT_SILU) return go(activate_kernel<float, ACT_SILU>, activate_kernel<__nv_bfloat16, ACT_SILU>);
    if (kind == ACT_GELU_SIDE) return go(activate_kernel<float, ACT_GELU_SIDE>, activate_kernel<__nv_bfloat16, ACT_GELU_SIDE>);
    return cudaErrorInvalidValue;
}

cudaError_t launch_rope_angles(const int* positions, const double* freqs, double magnitude, float2* out, int rows, int half, cudaStream_t st) {
    if (rows * half == 0) return cudaSuccess;
    rope_angles_kernel<<<(rows * half + 127) / 128, 128, 0, st>>>(positions, freqs, magnitude, out, rows, half);
    return cudaGetLastError();
}

cudaError_t launch_gemv_dense(const GemvDenseParams& p, cudaStream_t st) {
    if (p.act == ACT_SILU) return cudaErrorInvalidValue;
    if (p.m < 1 || p.m > 8 || p.n < 1 || p.k % 8 || p.ldw % 8 || p.w_z % 8 || p.x_row % 8 || p.x_z % 8 || (p.act != ACT_NONE && p.out_f32)) return cudaErrorInvalidValue;
    // split K until every warp has about eight blocks of 32 and the grid fills the machine
    const int blocks = (p.k + 31) / 32, tiles = (p.n + 15) / 16 * p.z;
    int wk = 1;
    while (wk < SKINNY_WARPS && blocks >= 16 * wk && (blocks > 64 * wk || tiles * wk < 148 * 32)) wk *= 2;
    const int cols = SKINNY_WARPS / wk * 16;
    const dim3 grid((p.n + cols - 1) / cols, p.z);
    auto go = [&](auto kernel) { return launch_pdl(kernel, grid, dim3(32 * SKINNY_WARPS), 0, st, p, wk); };
    if (p.act == ACT_GELU_MUL) return go(gemv_dense_kernel<ACT_GELU_MUL, __nv_bfloat16>);
    if (p.act == ACT_SILU_MUL) return go(gemv_dense_kernel<ACT_SILU_MUL, __nv_bfloat16>);
    if (p.act == ACT_GATE) return go(gemv_dense_kernel<ACT_GATE, __nv_bfloat16>);
    if (p.act == ACT_RELU2) return go(gemv_dense_kernel<ACT_RELU2, __nv_bfloat16>);
    if (p.act == ACT_GELU) return go(gemv_dense_kernel<ACT_GELU, __nv_bfloat16>);
    if (p.act == ACT_GELU_SIDE) return go(gemv_dense_kernel<ACT_GELU_SIDE, __nv_bfloat16>);
    return p.out_f32 ? go(gemv_dense_kernel<ACT_NONE, float>) : go(gemv_dense_kernel<ACT_NONE, __nv_bfloat16>);
}

LLM_DEFINE_BOUNDS_STATUS_READER(bounds_status_dense)

}  // namespace llm
