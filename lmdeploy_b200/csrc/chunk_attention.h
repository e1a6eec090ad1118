// Pieces of the chunk attention that its kernels share.
#pragma once
#include "mixers.h"
#include "numeric.cuh"

namespace tmb {

// first token that position i sees
__host__ __device__ __forceinline__ int chunk_first(int i, int chunk)
{
    return chunk > 0 ? i - i % chunk : 0;
}

// The 16-bit kernels hold a weight in fp16 times this, so that weights down to 2^-26 keep all their digits; outputs are
// divided by it at the end.
constexpr float kWeightScale = 4096.f;

struct ChunkKernelParams {
    ChunkAttention a;
    MixerCall      c;
};

// tcgen05 prefill (chunk_attention_tc.cu) and the fused one-token kernel (chunk_attention_decode.cu), bf16
bool chunk_attention_tc_supported(const ChunkAttention& a, const MixerCall& c);
int  chunk_attention_tc(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st);
bool chunk_attention_step_supported(const tm_handle* h, const ChunkAttention& a, const MixerCall& c);
int  chunk_attention_step(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st);

}  // namespace tmb
