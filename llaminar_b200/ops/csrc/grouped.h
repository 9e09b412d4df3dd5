// Launchers around grouped-query attention with per-head keys and values in the paged cache (the tensor-core kernels: ops.h).  `f32`
// selects the 32-bit build (activations and cache as float) instead of the bf16 one; norms, angles, scores, softmax and gates are 32-bit
// in both.  The projected rows may be float in the bf16 build as well (`in_f32`): decode steps keep their projections at accumulator
// precision.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stddef.h>

namespace llm {

// Projected rows [q | k | ...] -> queries RMS-normed over all heads, and the token's entry of the paged cache [pages, 2, kv heads, 64,
// dim]: keys RMS-normed over all heads, values as projected (tied: the keys before their norm).
struct AttnPrepParams {
    const void* in; size_t in_row; int q_off, k_off, v_off;      // v_off = k_off: tied values
    const float *q_norm, *k_norm;                                // [n_heads * dim], [n_kv_heads * dim]
    const int *positions, *seq_ids, *block_table;
    int max_pages, n_seqs, n_pages;
    void* q_out;                                                 // [T, n_heads, dim]
    void* kv;
    int n_heads, n_kv_heads, dim, true_dim;                      // padded head size, and the one that the means are taken over
    float eps;
};
cudaError_t launch_attn_prep(const AttnPrepParams& p, int rows, bool in_f32, bool f32, cudaStream_t st);

// Projected rows [q | k | v | ...] -> queries and keys RMS-normed per head (one gain per value, shared by the heads) and rotated, values as
// projected.  `dim` is the padded head size of all three; gains and rows are zero behind the true sizes.
struct HeadPrepParams {
    const void* in; size_t in_row; int q_off, k_off, v_off;
    const float *q_norm, *k_norm;                                // [dim]
    const float2* angles; int half;                              // [T, half]: pairs (i, i + half) turn, the rest passes
    const int *positions, *seq_ids, *block_table;
    int max_pages, n_seqs, n_pages;
    void* q_out;                                                 // [T, n_heads, dim]
    void* kv;
    int n_heads, n_kv_heads, dim, true_dim;                      // true_dim: what the means are taken over
    float eps;
};
cudaError_t launch_head_prep(const HeadPrepParams& p, int rows, bool in_f32, bool f32, cudaStream_t st);

// Attention of every row over the paged cache in float arithmetic, any size: the 32-bit mode, and shapes without a tensor-core kernel.
struct AttnPlainParams {
    const void* q; const void* kv; void* out;                    // [T, n_heads, dim], cache, [T, n_heads, dim]
    const int *positions, *seq_ids, *block_table;
    int max_pages, n_seqs, n_pages;
    int n_heads, n_kv_heads, dim, window;
    float scale;
    const float* sink;                                           // optional [n_heads]
    const void* gate; size_t gate_row; int gate_heads;           // optional, sigmoid; float if gate_f32; gate_heads: one number per head
    int chunk;                                                   // a row sees keys of its own chunk of positions only (0: no chunks)
    float softcap;                                               // scores s become softcap * tanh(s / softcap) (0: as they are)
};
cudaError_t launch_attn_plain(const AttnPlainParams& p, int rows, bool gate_f32, bool f32, cudaStream_t st);

int bounds_status_grouped(bool reset);

}  // namespace llm
