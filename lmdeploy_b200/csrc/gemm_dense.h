// Dense GEMM of the config-driven decoder: out[t, n] = sum_k x[t, k] * w[n, k], with the norm in front of it and the
// elementwise work behind it in the epilogue.  bf16 operands run on the tcgen05 tensor core (fp32 accumulation), fp32
// operands on the CUDA cores in true fp32.
#pragma once
#include "handle.h"

#include <cuda.h>
#include <cuda_runtime.h>

namespace tmb {

enum class DenseKind : int {
    kStore,     // out[t][n] in the element type
    kF32,       // out[t][n] in fp32
    kInput,     // a layer's input projections: columns [0, split) are stored in the element type (those in
                // [tanh_lo, tanh_hi) through tanh); from `split` on, columns come in (gate, up) pairs and
                // act[t][(n - split) / 2] = activation(gate, up)
    kResidual,  // residual[t][n] += y (fp32), or += mult * sigmoid(gate[t][n] + gate_bias[n]) * y where there is a gate;
                // optionally also cast[t][n] = residual in the element type and the tile's part of the row's sum of squares
};

enum class DenseActivation : int {
    kGeluTanh,      // gelu_tanh(gate) * up
    kClampedSwish,  // g = min(gate, limit), u = clamp(up, -limit, limit): g * sigmoid(slope * g) * (u + 1)
};

struct DenseEpilogue {
    DenseKind kind = DenseKind::kStore;
    // rows scaled by gain / sqrt(sum of squares / width + eps): RMS norm of x with one gain for all coordinates, applied
    // behind the product.  The sum of squares comes in `ssq_parts` parts, [part][ssq_stride]; null = no scaling.
    const float* ssq = nullptr;
    int          ssq_parts = 0, ssq_stride = 0;
    float        inv_width = 0.f, eps = 0.f;
    const float* gain = nullptr;

    void* out     = nullptr;
    int   out_ld  = 0;
    int   tanh_lo = 0, tanh_hi = 0, split = 0;
    void* act     = nullptr;
    int   act_ld  = 0;
    DenseActivation activation = DenseActivation::kGeluTanh;
    float           limit = 0.f, slope = 0.f;
    // kStore, kInput: columns from f32_from on go to f32_out[t][n - f32_from] in fp32 instead (0: none)
    float* f32_out  = nullptr;
    int    f32_from = 0, f32_ld = 0;

    float* residual    = nullptr;
    int    residual_ld = 0;
    void*  cast        = nullptr;
    int    cast_ld     = 0;
    float* ssq_out     = nullptr;  // [column tile of 128][ssq_out_stride]
    int    ssq_out_stride = 0;
    const void*  gate      = nullptr;
    int          gate_ld   = 0;
    const float* gate_bias = nullptr;
    float        mult      = 1.f;
};

// Products of several row groups, each with a weight of its own (the experts of a mixture): group g's rows are
// [offsets[g], offsets[g + 1]) of x and of the output, its weight rows [g * n_out, (g + 1) * n_out) of w.  The offsets are
// read on the device; `tokens` of the call is an upper bound on offsets[groups].
struct DenseGroups {
    int        count   = 0;  // 0: a plain product
    const int* offsets = nullptr;
};
constexpr int kMaxDenseGroups = 1024;

struct DenseGemm {
    const void* w = nullptr;  // [n_out][ldw]
    const void* x = nullptr;  // [tokens][ldx]
    int         ldw = 0, ldx = 0;
    int         tokens = 0, n_out = 0, k = 0;
    // output columns from x2_from on (a multiple of kDenseTile; 0: none) are products with x2 instead, rows as far apart as x's
    const void* x2      = nullptr;
    int         x2_from = 0;
    DenseGroups   groups;
    DenseEpilogue ep;
};

constexpr int kDenseTile = 128;  // output columns of one tile: the granularity of `split` and of ssq_out

// bf16: ldw and ldx multiples of 8, 16-byte aligned bases.  Scratch and tickets come from the handle.
int dense_gemm(tm_handle* h, const DenseGemm& g, bool f32, cudaStream_t st, bool pdl);

}  // namespace tmb
