// Launchers of the mixers with a recurrent state.  `f32` selects the 32-bit build (activations and
// cache as float) instead of the bf16 one; norms, gates and state are 32-bit in both.  The projected rows may be
// float in the bf16 build as well (`in_f32`): decode steps keep their projections at accumulator precision.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stddef.h>

namespace llm {

// Linear attention with a recurrent state per head: mLSTM (with `gates`), or a fixed decay (retention, lightning attention).
struct LinearParams {
    const void* in; size_t in_row;                               // projected rows; head h of q starts at q_off + h * dim
    int q_off, k_off, v_off, g_off;
    const float* gates; size_t gate_row;                         // [T][log input gates, then log forget gates, of all heads] before bias and cap
    const float *bias_i, *bias_f;                                // [heads]
    float cap;
    const float* decay;                                          // [heads]
    const float2* angles; int half;                              // rotation of q and k (half = 0: none)
    float q_scale, k_scale;
    const int* cu;                                               // [n_seqs + 1] rows of the sequences (nullptr: one row each)
    const int *positions, *slots;                                // [T], [n_seqs]
    float *S, *n, *m;                                            // [slots, heads, vdim, dim], [slots, heads, dim], [slots, heads]
    int n_slots, heads, dim, vdim, true_vdim;                    // padded to multiples of 8
    const float* norm_w;                                         // optional [heads * vdim]
    int silu;                                                    // output gate: silu or sigmoid
    int silu_in;                                                 // q, k and v pass through silu first (row-wise kernel; the chunk kernels want them so)
    int raw;                                                     // o as it is, without norm and gate (`g_off` unused)
    void* out; size_t out_row;                                   // [T, heads * vdim]
    float eps;
};
// row after row: decode steps, the 32-bit mode, sizes without a chunk kernel
cudaError_t launch_linear_rows(const LinearParams& p, int n_seqs, bool in_f32, bool f32, cudaStream_t st);
// Chunk-parallel form for prompts: bf16 rows, heads of at most 128 key values (linear_tc.cu).  Sequences are cut into chunks of
// LINEAR_CHUNK rows; `chunks` holds (first row, rows, sequence, 0) of each, `seqs` (first chunk, chunks, 0, 0).  Scratch: state
// [chunks][heads][vdim][dim] float, vec [chunks][heads][dim] float, scal [chunks][heads][4] float, gate [chunks][heads][LINEAR_CHUNK].  o
// [T, heads * vdim] bf16: the heads' outputs before norm and gate, where a head of more than 256 values is spread over CTAs.
constexpr int LINEAR_CHUNK = 128;
struct LinearChunks {
    const int4 *chunks, *seqs;
    int n_chunks, n_seqs, rows;
    float *state, *vec, *scal;
    float4* gate;                                                // mLSTM: what the gates of every row come to, chunk_state to chunk_out
    __nv_bfloat16* o;
    int* status;                                                 // receives STATUS_TIMEOUT if a wait gave up
};
bool linear_chunk_fits(int dim, int vdim);
cudaError_t launch_linear_chunk(const LinearParams& p, const LinearChunks& c, cudaStream_t st);
// out[t, h] = o[t, h] / rms(o[t, h]) * norm_w * gate(in[t, g_off + ...]), bf16
cudaError_t launch_head_gate(const LinearParams& p, const __nv_bfloat16* o, int rows, cudaStream_t st);

// out[t] = o[t] / rms(o[t]) * norm_w * sigmoid(in[t, g_off + ...]): norm over all heads' n values together, `true_n` of them not padding.
struct JointGateParams {
    const void* o; size_t o_row;                                 // float or bf16, as `in`
    const void* in; size_t in_row; int g_off;
    const float* norm_w;                                         // [n]
    void* out; size_t out_row;
    int n, true_n;
    float eps;
};
cudaError_t launch_joint_gate(const JointGateParams& p, int rows, bool in_f32, bool f32, cudaStream_t st);

int bounds_status_mixers(bool reset);
int bounds_status_linear_tc(bool reset);

}  // namespace llm
