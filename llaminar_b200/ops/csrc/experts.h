// Launchers of mixture-of-experts feed-forwards with unquantised matrices.  `f32` selects the 32-bit build (activations and weights as
// float) instead of the bf16 one; router logits, the choice and its weights are 32-bit in both.  A pair is (token, one of its chosen
// experts): pair p belongs to token p / top.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stddef.h>

namespace llm {

constexpr int EXPERTS_MAX_TOP = 32, EXPERTS_MAX = 1024;

// Router logits x W^T + bias (or given in `logits`), the `top` largest of them (the lower expert first when equal) and the softmax over
// just those (what dividing their part of a softmax over all experts by its sum gives).  With `groups` > 1 the experts form that many
// groups of neighbours, and only those of the `keep` groups with the largest logits (the lower group first when equal) can be chosen.
// With `counts` (zeroed by the caller) the pairs of every expert are counted and numbered.
struct ExpertRouteParams {
    const void* x; size_t x_row;                   // [T, d]
    const void* router;                            // [n, d]
    const float* logits;                           // [T, n] without bias, or nullptr
    const float* bias;                             // [n]
    int* ids; float* weights;                      // [T, top]
    int *counts, *ranks;                           // [n], [T * top]: number of a pair among those of its expert
    int d, n, top, groups, keep;
};
cudaError_t launch_expert_route(const ExpertRouteParams& p, int rows, bool f32, cudaStream_t st);

// Rows of x sorted by expert: pair p goes to row place[p] of xs.
struct ExpertPlaceParams {
    const __nv_bfloat16* x; size_t x_row;          // [T, d]
    const int *ids, *ranks, *counts;
    int* place;                                    // [T * top]
    __nv_bfloat16* xs;                             // [T * top, d]
    int d, n, top;
};
cudaError_t launch_expert_place(const ExpertPlaceParams& p, int rows, cudaStream_t st);

// out[pair] = x[pair / div] W_e^T with e = ids[pair]; `pair_act`: W_e stacks gate and up, out = silu(gate) * up, or with a `limit` g
// sigmoid(1.702 g) (u + 1) of g = min(gate, limit) and u = up clamped to [-limit, limit].
struct ExpertRowsParams {
    const void* w;                                 // [experts, n (pair_act: 2n), k]
    const void* x; size_t x_row;
    const int* ids;                                // [pairs]
    void* out;                                     // [pairs, n]
    int pairs, div, n, k, experts;
    bool pair_act;
    float limit;
};
// few pairs, bf16: the weights of every chosen expert are read once for all of its pairs (in groups of 8 to 32)
constexpr int EXPERT_ROWS_MAX_PAIRS = 1024;
cudaError_t launch_expert_rows(const ExpertRowsParams& p, cudaStream_t st);
// float arithmetic, any number of pairs and any size
cudaError_t launch_expert_plain(const ExpertRowsParams& p, bool f32, cudaStream_t st);

// The same for pairs sorted by expert (tcgen05): rows [offset of e, + counts[e]) of x and out belong to expert e.
struct ExpertGroupedParams {
    const int* counts;
    __nv_bfloat16* out;                            // [pairs, n]
    int pairs, n, k, experts;
    float limit;
};
bool expert_grouped_fits(int n, int k, int experts);
cudaError_t launch_expert_grouped(const __nv_bfloat16* w, const __nv_bfloat16* x, const ExpertGroupedParams& p, bool pair_act, int* status, cudaStream_t st);

int bounds_status_experts(bool reset);

}  // namespace llm
