// Pieces of the window attention that its kernels share.
#pragma once
#include "mixers.h"
#include "numeric.cuh"

namespace tmb {

// What position i sees: pooled blocks [0, blocks), then tokens [first, i]
struct Visible {
    int first, blocks;
};
__host__ __device__ __forceinline__ Visible visible_of(int i, int window, int pool)
{
    Visible v{0, 0};
    if (window > 0) {
        const int out = i - window + 1;  // tokens that have left the window
        if (out > 0) {
            v.first = out;
            if (pool > 0) v.blocks = out / pool;
        }
    }
    return v;
}

struct WindowKernelParams {
    WindowAttention a;
    MixerCall       c;
};

// tcgen05 prefill attention (window_attention_tc.cu): bf16, q rotated, keys / values / pooled rows in the slab
bool window_attention_tc_supported(const WindowAttention& a, const MixerCall& c);
int  window_attention_tc(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st);
// one-token attention with the rotation, the cache append and the pooling fused in (window_attention_decode.cu): bf16
bool window_attention_step_supported(const WindowAttention& a, const MixerCall& c);
int  window_attention_step(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st);

}  // namespace tmb
