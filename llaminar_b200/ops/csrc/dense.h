// Launchers of what models with unquantised matrices share: fused norms of the residual stream, activations, rotary angles and
// the small-batch matrix product.  `f32` selects the 32-bit build of a kernel (activations as float) instead of the bf16 one;
// residual stream, norms and angles are 32-bit in both.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stddef.h>

namespace llm {

// v = y[row(t)], or the sum of y[row(t, j)] * y_w[t, j] over j < n_parts, or half the sum of RMSNorm(y[t]) * w_y and RMSNorm(y2[t]) * w_y2
// h[t] = (add ? h[t] : 0) + (norm of v) * w_post, or v * factor ; xn[t] = (norm of h[t]) * w_next ; copies of h[t] in the activation type
struct ResidNormParams {
    const void* y;                 // activation type; nullptr: h is only read
    size_t y_stride;
    const int* y_rows;             // optional gather (embedding lookup, sorted experts): row(t) = y_rows[t], row(t, j) = y_rows[t * n_parts + j]
    int n_y_rows;                  // rows of y (bounds-check build)
    const float* y_w;              // with n_parts > 0: weights of the parts (chosen experts)
    int n_parts;
    const void* y2;                // optional second sublayer output [T, d]
    size_t y2_stride;
    const float *w_y, *w_y2;       // [d], with y2
    const float* w_post;           // [d]; nullptr: no norm, v * factor
    float factor;
    int center_post, center_next;  // the norm takes the mean off first
    float* h;                      // [T, d]
    int add;
    const float* w_next;           // optional [d]
    void* xn;                      // [T, d]
    void *copy0, *copy1;           // optional
    size_t copy_stride;
    int d;
    float eps;
};
cudaError_t launch_resid_norm(const ResidNormParams& p, int rows, bool f32, cudaStream_t st);

// One residual update of layers whose sublayers run side by side, the weighted sum over depth behind it, and the norms that follow:
// x = (add ? h[t] : 0) + y[row(t)] + z[row(t)], or z's weighted sum of rows as in ResidNormParams
// h[t] = w[n_past] * x + sum over j < n_past of w[j] * past[j][t]  (w nullptr: x), past[n_past][t] = x if `keep`
// xn0[t] = (RMSNorm of h[t]) * gain0, xn1[t] the same with gain1
struct DepthMixParams {
    const void *y, *z;             // activation type; both nullptr (and n_past = 0): h is only read
    size_t y_stride, z_stride;
    const int *y_rows, *z_rows;    // optional gather (embedding and position tables, sorted experts)
    int n_y_rows, n_z_rows;        // rows of y and z (bounds-check build)
    const float* z_w;              // with n_parts > 0: weights of the parts (chosen experts)
    int n_parts;
    float* h;                      // [T, d]
    int add;
    float* past;                   // streams of [T, d], `past_stride` values apart
    size_t past_stride;
    int n_past, keep;
    const float* w;                // [n_past + 1]
    const float *gain0, *gain1;    // optional: one gain per value, or (gain_step = 0) one for all
    int gain_step;
    void *xn0, *xn1;               // [T, d]
    int d;
    float eps;
};
cudaError_t launch_depth_mix(const DepthMixParams& p, int rows, bool f32, cudaStream_t st);

// Activations behind a product.  GELU_MUL: gelu_tanh(first half of the columns) * second half, SILU_MUL the same with silu; RELU2: squared
// relu; GELU, SILU: without a second half; GELU_SIDE: gelu_tanh times the token's row of a table (columns [0, side_cols), zero behind);
// GATE: times the sigmoid of the row's own row of the table (tokens unused).
enum Activation : int { ACT_NONE = 0, ACT_GELU_MUL = 1, ACT_RELU2 = 2, ACT_GELU_SIDE = 3, ACT_SILU_MUL = 4, ACT_GATE = 5, ACT_GELU = 6, ACT_SILU = 7 };
constexpr bool act_pairs(int act) { return act == ACT_GELU_MUL || act == ACT_SILU_MUL; }
struct SideTable { const void* table; size_t row; int cols, n_rows; const int* tokens; };
// act[t, 0..n) from x[t, 0..n) (GELU_MUL, SILU_MUL: 2n columns); rows x_row and act_row values apart
cudaError_t launch_activate(const void* x, size_t x_row, void* act, size_t act_row, int rows, int n, int kind, const SideTable& side, bool f32, cudaStream_t st);

// out[t, i] = magnitude * (cos, sin)(positions[t] * freqs[i])
cudaError_t launch_rope_angles(const int* positions, const double* freqs, double magnitude, float2* out, int rows, int half, cudaStream_t st);

// out[z][m, :] = act(x[z][m, :] W[z]^T) for up to 8 rows, bf16 weights.  GELU_MUL, SILU_MUL: W holds 2n rows.  GATE: the table's row m
// holds the gates of all z, n columns each.
struct GemvDenseParams {
    const __nv_bfloat16* w; size_t w_z; int ldw;
    const __nv_bfloat16* x; size_t x_row, x_z;
    void* out; size_t o_row, o_z;
    int n, k, m, z;
    bool out_f32;
    int act;                       // with one: out is bf16
    SideTable side;
};
cudaError_t launch_gemv_dense(const GemvDenseParams& p, cudaStream_t st);

int bounds_status_dense(bool reset);

}  // namespace llm
