// Mixture of experts: routing, and the movement of token rows to their experts and back.  The experts themselves are two
// grouped products (DenseGroups in gemm_dense.h) over rows sorted by expert.
#pragma once
#include "handle.h"

#include <cuda_runtime.h>

namespace tmb {

// Scores are a softmax over all router outputs; `top` of them are chosen by score + correction, out of the `keep` groups
// (of `groups` equal groups of neighbours) whose best choice score is highest; the weights are the scores as they are.
// The last `identity` outputs stand for experts that give back their input.
struct MoeRouter {
    int          experts = 0, identity = 0, top = 0, groups = 1, keep = 1;
    const float* correction = nullptr;  // [experts + identity]
    __host__ __device__ int outputs() const { return experts + identity; }
};
constexpr int kMaxRouterOutputs = 1024, kMaxRouterTop = 32;

// Device buffers of one pass
struct MoeRows {
    int*   counts  = nullptr;  // [experts], zero before a dispatch; the rows kernel behind the layer clears it again
    int*   offsets = nullptr;  // [experts + 1] first row of every expert
    int*   slots   = nullptr;  // [tokens][top] row of a chosen expert, -1: identity
    float* weights = nullptr;  // [tokens][top]
    int*   ranks   = nullptr;  // [tokens][top] scratch
    void*  sorted  = nullptr;  // [tokens * top][ld] input rows in expert order
    int    ld      = 0;
};

// router logits [tokens][logits_ld] (fp32) and input rows [tokens][rows.ld] -> offsets, slots, weights, sorted
int moe_dispatch(tm_handle* h, const MoeRouter& r, const MoeRows& m, const float* logits, int logits_ld, const void* input, int tokens, int width,
                 bool f32, cudaStream_t st, bool pdl);

// What stands between two layers with vector norms: the embedding of a first layer, or the feed-forward's contribution to
// the residual, then the norms of the next layer (or of the output).  One CTA per token.
struct RowsCall {
    float* x      = nullptr;  // [tokens][width] residual
    int    tokens = 0, width = 0;
    // x = embed[ids] (first layer)
    const void* embed = nullptr;
    const int*  ids   = nullptr;
    int         vocab = 0;
    // x += mult * sigmoid(gate + gate_bias) * sum of weights * (expert rows, or `input` for identity)
    const void*  expert_rows = nullptr;  // [row][width]; null: no feed-forward
    const void*  input       = nullptr;  // [tokens][input_ld]
    int          input_ld    = 0;
    const int*   slots       = nullptr;
    const float* weights     = nullptr;
    int          top         = 0;
    const void*  gate        = nullptr;
    int          gate_ld     = 0;
    const float* gate_bias   = nullptr;
    float        mult        = 1.f;
    // out_a = norm(x) * weight_a, out_b likewise (null: not wanted), [tokens][out_ld] in the element type
    const float *weight_a = nullptr, *weight_b = nullptr;
    void *       out_a = nullptr, *out_b = nullptr;
    int          out_ld = 0;
    float        eps    = 0.f;
    int*         clear  = nullptr;  // ints set to zero by the first CTA
    int          clear_count = 0;
};
int norm_rows(tm_handle* h, const RowsCall& c, bool f32, cudaStream_t st, bool pdl);

}  // namespace tmb
