// Kernels around the layers of a decode step (step_kernels.h).
#include "step_kernels.h"

#include <cmath>
#include <cstdint>

namespace tmb {
namespace {

// greedy pick over logits laid out [tp][B][vocab / tp]; ties go to the lowest token id
__global__ void argmax_kernel(const float* logits, int* picked, int* output_ids, const int* step,
                              const unsigned char* inactive, int B, int local_vocab, int tp, int max_steps)
{
    __shared__ float s_val[1024];
    __shared__ int   s_idx[1024];
    const int b    = blockIdx.x;
    float     best = -INFINITY;
    int       idx  = 0x7fffffff;
    auto take = [&](float x, int i) {
        if (x > best || (x == best && i < idx)) {
            best = x;
            idx  = i;
        }
    };
    for (int r = 0; r < tp; ++r) {
        const float* row = logits + ((size_t)r * B + b) * local_vocab;
        if ((local_vocab & 3) == 0 && (reinterpret_cast<uintptr_t>(row) & 15) == 0) {
            // four logits per load, several loads in flight per thread
            const float4* row4 = reinterpret_cast<const float4*>(row);
            for (int v = threadIdx.x; v < local_vocab / 4; v += blockDim.x) {
                const float4 x = row4[v];
                const int    i = r * local_vocab + 4 * v;
                take(x.x, i);
                take(x.y, i + 1);
                take(x.z, i + 2);
                take(x.w, i + 3);
            }
        }
        else {
            for (int v = threadIdx.x; v < local_vocab; v += blockDim.x) take(row[v], r * local_vocab + v);
        }
    }
    s_val[threadIdx.x] = best;
    s_idx[threadIdx.x] = idx;
    __syncthreads();
    for (int off = blockDim.x / 2; off > 0; off >>= 1) {
        if (threadIdx.x < off) {
            const float x = s_val[threadIdx.x + off];
            const int   i = s_idx[threadIdx.x + off];
            if (x > s_val[threadIdx.x] || (x == s_val[threadIdx.x] && i < s_idx[threadIdx.x])) {
                s_val[threadIdx.x] = x;
                s_idx[threadIdx.x] = i;
            }
        }
        __syncthreads();
    }
    if (threadIdx.x == 0) {
        const int s = *step;
        if (!inactive[b]) {
            picked[b] = s_idx[0];
        }
        if (s < max_steps) {
            output_ids[(size_t)s * B + b] = inactive[b] ? -1 : s_idx[0];
        }
    }
}

__global__ void advance_kernel(int* step, int* lengths, const unsigned char* inactive, int B)
{
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b < B && !inactive[b]) lengths[b] += 1;
    if (b == 0) *step += 1;
}

}  // namespace

cudaError_t step_argmax(const float* logits, int* picked, int* output_ids, const int* step, const unsigned char* inactive, int B,
                        int local_vocab, int tp, int max_steps, cudaStream_t st)
{
    argmax_kernel<<<B, 1024, 0, st>>>(logits, picked, output_ids, step, inactive, B, local_vocab, tp, max_steps);
    return cudaPeekAtLastError();
}

cudaError_t step_advance(int* step, int* lengths, const unsigned char* inactive, int B, cudaStream_t st)
{
    advance_kernel<<<(B + 127) / 128, 128, 0, st>>>(step, lengths, inactive, B);
    return cudaPeekAtLastError();
}

}  // namespace tmb
