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

// Projected rows [q | k | v | ...] -> a causal convolution over time on each of their channels, then queries and keys rotated (pairs (i, i +
// half)), queries times their head's temperature, values mixed with those of an earlier layer; appended to the cache like above.  The
// last taps - 1 rows of a sequence come from `ring` [slots, taps, channels] (position p in place p mod taps, channels = (n_heads + 2
// n_kv_heads) * dim).  One row per sequence (`cu` nullptr): the row enters the ring here; portions leave it to launch_conv_keep.
struct ConvPrepParams {
    const void* in; size_t in_row;                               // channels [0, (n_heads + 2 n_kv_heads) * dim) of a row
    const float* taps; int n_taps;                               // [n_taps][channels], the newest tap last
    float* ring; const int* slots; int n_slots;                  // [n_seqs]
    const int* cu;                                               // [n_seqs + 1] first rows of the sequences, or nullptr
    const float2* angles; int half;                              // [T, half] (half = 0: no rotation)
    const float* q_gain;                                         // optional [n_heads]
    float* first; int first_dim;                                 // optional [T, n_kv_heads, first_dim]: values of the earlier layer
    const float* share;                                          // v = (1 - share) v + share first; nullptr: `first` receives v
    const int *positions, *seq_ids, *block_table;
    int max_pages, n_seqs, n_pages;
    void* q_out;                                                 // [T, n_heads, dim]
    void* kv;
    int n_heads, n_kv_heads, dim, rows;
};
cudaError_t launch_conv_prep(const ConvPrepParams& p, bool in_f32, bool f32, cudaStream_t st);
// the last rows of every portion into the ring (`cu` given)
cudaError_t launch_conv_keep(const ConvPrepParams& p, bool in_f32, cudaStream_t st);

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
