// Launchers of the kernels around latent attention (low-rank key/value cache shared by all heads).  `f32` selects the 32-bit
// build of a kernel (activations and cache as float) instead of the bf16 one; angles, norms, scores and softmax are 32-bit in both.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stddef.h>

namespace llm {

// Down projection row [q latent | kv latent | rotated key] -> normed query latent, and the token's cache row
// [normed kv latent, padded to rot_off | rotated key part, padded to width].
struct LatentPrepParams {
    const void* down; size_t down_stride;
    const float *q_norm, *kv_norm;
    const float2* angles; int half;            // [T, half]
    const int *positions, *seq_ids, *block_table;
    int max_pages, n_seqs, n_pages;
    void* cq; size_t cq_stride;                // [T, cq_stride], columns behind q_rank are zeroed
    void* kv;                                  // [n_pages, 64, width]
    int q_rank, kv_rank, rot_dim, rot_off, width;
    float eps;
};
cudaError_t launch_latent_prep(const LatentPrepParams& p, int rows, bool f32, cudaStream_t st);

// Attention of single rows, each with its own sequence and position, over the latent cache: queries are already multiplied
// into the latent space, the result is the weighted sum of latents per head.
struct LatentRowsParams {
    const void* q_lat; size_t ql_row, ql_head; // [row z][head][kv_rank padded to rot_off]
    const void* q; size_t q_row, q_head;       // [token][head] up-projected query; its rotated part starts at q_rot_off
    int q_rot_off;
    const float2* angles; int half;
    const int* rows;                           // token of row z (nullptr: z)
    const int *positions, *seq_ids, *block_table;
    int max_pages, n_seqs, n_pages;
    const void* kv;                            // [n_pages, 64, width]
    int width, rot_off, rot_dim;
    int n_heads, window;
    float scale;
    const float* sink;                         // optional [n_heads]
    void* out; size_t out_row, out_head;       // [row z][head][rot_off]
    float *part_o, *part_ml;                   // [rows * head groups * splits][group][rot_off], [...][group][2]
};
cudaError_t launch_latent_rows(const LatentRowsParams& p, int rows, int n_splits, bool f32, bool plain, cudaStream_t st);
// whether the mma.sync kernel takes these sizes (otherwise, or with `plain`, launch_latent_rows runs the plain kernel)
bool latent_rows_has_kernel(int width, int rot_off);
// tcgen05 form: heads per CTA (the group of the split scratch), 0 where the sizes do not fit
int latent_rows_tc_heads(int width, int rot_off, int rot_dim, int n_heads);
cudaError_t launch_latent_rows_tc(const LatentRowsParams& p, int rows, int n_splits, int* status, cudaStream_t st);
// merges the splits of either form
cudaError_t launch_latent_merge(const LatentRowsParams& p, int rows, int n_splits, int group, cudaStream_t st);

// Cache rows of the sequences' visible keys -> contiguous rows: buffer row k_off[s] + i holds position k_pos0[s] + i.
struct LatentSeq { int seq, q_start, q_len, q_pos0, k_off, k_pos0, k_len, pad; };
cudaError_t launch_latent_gather(const void* kv, const LatentSeq* seqs, int n, int max_k_len, const int* block_table, int max_pages,
                                 int n_pages, int width, void* out, bool f32, cudaStream_t st);

// Attention of prompt chunks with keys and values written out per head.
struct LatentChunkParams {
    const __nv_bfloat16* q; size_t q_row, q_head;      // [token][head][dim | rot]
    const float2* angles; int half;
    const __nv_bfloat16* k;                            // [key][head][dim]
    const __nv_bfloat16* v;                            // [key][head][vdim]; tcgen05 form: [head][vdim][key]
    const __nv_bfloat16* lat; size_t lat_row; int rot_off;
    const LatentSeq* seqs;
    __nv_bfloat16* out; size_t out_row;                // [token][head * vdim]
    int dim, rot, vdim, n_heads, window;               // padded to multiples of 8
    float scale;
    const float* sink;
    const __nv_bfloat16* gate; size_t gate_row;        // optional [token][head * vdim]: the result times its sigmoid (rows of whole 16-byte units)
};
cudaError_t launch_latent_chunk(const LatentChunkParams& p, int n_seqs, int max_q_len, cudaStream_t st);
bool latent_chunk_has_kernel(int dk, int dv);
// tcgen05 form; n_keys (a multiple of 8, as every k_off) rows of k and lat, columns of v.  `status` receives STATUS_TIMEOUT if a wait gave up.
cudaError_t launch_latent_chunk_tc(const LatentChunkParams& p, int n_keys, int n_seqs, int max_q_len, int* status, cudaStream_t st);
bool latent_chunk_tc_fits(int dim, int rot, int vdim);

int bounds_status_latent(bool reset);
int bounds_status_latent_tc(bool reset);

}  // namespace llm
