// Building blocks shared by the tcgen05 kernels whose operand tiles arrive by TMA (latent_tc.cu, linear_tc.cu): swizzled tiles,
// rotation of 16-byte units, tensor-memory loads and stores, tensor maps.
#pragma once
#include "tc_common.cuh"

namespace llm {
namespace tc5 {

constexpr float LOG2E = 1.4426950408889634f;
constexpr int ATOM = 128 * 128;                    // 128 rows x 64 bf16: one swizzled operand atom

LLM_DEVICE float ex2(float x) {                    // 2^x, approximate; -inf -> 0
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// 16-byte unit `unit` (0..7) of row `row` inside one operand atom
LLM_DEVICE uint32_t atom_addr(uint32_t base, int row, int unit) { return base + row * 128 + (((unit ^ row) & 7) << 4); }
LLM_DEVICE void st_shared_v4(uint32_t dst, const uint4& v) {
    asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};" ::"r"(dst), "r"(v.x), "r"(v.y), "r"(v.z), "r"(v.w) : "memory");
}
LLM_DEVICE void tmem_st32(uint32_t taddr, const uint32_t (&r)[32]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,"
                 "%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
                   "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
                   "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
                   "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31]) : "memory");
}
LLM_DEVICE void tmem_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// value i of a rotated part: pairs (i, i + half) turn, the rest passes
LLM_DEVICE float rotated(const __nv_bfloat16* x, int i, const float2* ang, int half) {
    const float v = __bfloat162float(x[i]);
    if (i < half) return v * ang[i].x - __bfloat162float(x[i + half]) * ang[i].y;
    if (i < 2 * half) return v * ang[i - half].x + __bfloat162float(x[i - half]) * ang[i - half].y;
    return v;
}
// values i0 .. i0 + 7 of it, zero from `n` on
LLM_DEVICE uint4 rotated8(const __nv_bfloat16* x, int i0, int n, const float2* ang, int half) {
    float v[8];
    if (half % 8 == 0 && i0 + 8 <= 2 * half) {                 // eight whole pairs: vector loads
        const bool first = i0 < half;
        const int a0 = first ? i0 : i0 - half;
        const uint4 own = *reinterpret_cast<const uint4*>(x + i0), other = *reinterpret_cast<const uint4*>(x + (first ? i0 + half : i0 - half));
        const uint32_t a[4] = {own.x, own.y, own.z, own.w}, b[4] = {other.x, other.y, other.z, other.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float4 cs = *reinterpret_cast<const float4*>(ang + a0 + 2 * j);       // cos, sin of two pairs
            const float s0 = first ? -cs.y : cs.y, s1 = first ? -cs.w : cs.w;
            v[2 * j] = bf16_lo(a[j]) * cs.x + bf16_lo(b[j]) * s0;
            v[2 * j + 1] = bf16_hi(a[j]) * cs.z + bf16_hi(b[j]) * s1;
        }
    } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = i0 + j < n ? rotated(x, i0 + j, ang, half) : 0.f;
    }
    return make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}

LLM_DEVICE void teardown(volatile int* abort_flag, int tid, int* status) {
    if (abort_flag[0]) {
        if (tid == 0 && status) atomicExch(status, (int)STATUS_TIMEOUT);
        for (int i = 0; i < 2000; ++i) __nanosleep(100);      // let copies still in flight land before the memory is reused
        __syncthreads();
    }
}

// MN-major, 128-byte swizzle: rows of 64 values along M, one row per k; 8-row groups 1024 bytes apart, 64-value groups `lead` apart
LLM_DEVICE uint64_t smem_desc_mn_sw128(uint32_t addr, uint32_t lead) {
    return (smem_desc_sw128(addr) & ~((uint64_t)0x3fff << 16)) | ((uint64_t)((lead >> 4) & 0x3fff) << 16);
}

template <int N> LLM_DEVICE void tmem_ld_n(uint32_t taddr, uint32_t (&r)[N]);
template <> LLM_DEVICE void tmem_ld_n<32>(uint32_t taddr, uint32_t (&r)[32]) { tmem_ld32_issue(taddr, r); tmem_wait_ld(r); }
template <> LLM_DEVICE void tmem_ld_n<16>(uint32_t taddr, uint32_t (&r)[16]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
                   "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]) : "r"(taddr));
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 16; ++i) asm volatile("" : "+r"(r[i]));
}
template <int N> LLM_DEVICE void tmem_st_n(uint32_t taddr, const uint32_t (&r)[N]);
template <> LLM_DEVICE void tmem_st_n<32>(uint32_t taddr, const uint32_t (&r)[32]) { tmem_st32(taddr, r); }
template <> LLM_DEVICE void tmem_st_n<16>(uint32_t taddr, const uint32_t (&r)[16]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
                   "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}
typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                  const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static EncodeTiledFn encode_fn() {
    static EncodeTiledFn fn = nullptr;
    if (!fn) {
        void* ptr = nullptr;
        cudaDriverEntryPointQueryResult qres;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres) == cudaSuccess && qres == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiledFn>(ptr);
    }
    return fn;
}
// bf16 matrix [rows, cols] with the given row stride (elements); boxes of 64 columns x box_rows rows, 128-byte swizzle
static bool make_map(CUtensorMap* m, const void* ptr, uint64_t cols, uint64_t rows, uint64_t stride, uint32_t box_rows) {
    EncodeTiledFn enc = encode_fn();
    if (!enc || (reinterpret_cast<uintptr_t>(ptr) & 15) || stride % 8) return false;
    const cuuint64_t dims[2] = {cols, rows}, strides[1] = {stride * 2};
    const cuuint32_t box[2] = {64, box_rows}, estr[2] = {1, 1};
    return enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
               CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
// bf16 tensor of N dimensions, the innermost dense; 128-byte swizzle, boxes of `box` elements, zeros outside
template <int N> static bool make_map_nd(CUtensorMap* m, const void* ptr, const cuuint64_t (&dims)[N], const cuuint64_t (&strides)[N - 1], const cuuint32_t (&box)[N]) {
    EncodeTiledFn enc = encode_fn();
    if (!enc || (reinterpret_cast<uintptr_t>(ptr) & 15)) return false;
    cuuint64_t bytes[N - 1];
    cuuint32_t estr[N];
    for (int i = 0; i < N; ++i) estr[i] = 1;
    for (int i = 0; i < N - 1; ++i) {
        if (strides[i] % 8) return false;
        bytes[i] = strides[i] * 2;
    }
    return enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, N, const_cast<void*>(ptr), dims, bytes, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
               CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
template <class K> static cudaError_t raise_smem(K kernel, size_t bytes) {
    return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

}  // namespace tc5
}  // namespace llm
