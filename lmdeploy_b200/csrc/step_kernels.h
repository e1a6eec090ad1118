// Kernels around the layers of a decode step that every model shares: greedy pick, step / length update.
#pragma once
#include <cuda_runtime.h>

namespace tmb {

// greedy pick over logits laid out [tp][B][local_vocab]; ties go to the lowest token id; inactive sequences keep their pick
cudaError_t step_argmax(const float* logits, int* picked, int* output_ids, const int* step, const unsigned char* inactive, int B,
                        int local_vocab, int tp, int max_steps, cudaStream_t st);
// lengths of active sequences and the step counter go up by one
cudaError_t step_advance(int* step, int* lengths, const unsigned char* inactive, int B, cudaStream_t st);

#ifdef __CUDACC__
// The input token of sequence b in this step, and whether it sits the step out
__device__ __forceinline__ int step_input(const int* step, const int* start_step, const int* forced_ids, const int* picked, int b, int B,
                                          int max_steps, int vocab, bool* off)
{
    const int s = *step;
    *off        = s >= max_steps || (start_step != nullptr && s < start_step[b]);
    int id      = picked[b];
    if (!*off && forced_ids != nullptr) {
        const int f = forced_ids[(size_t)s * B + b];
        if (f >= 0) id = f;
    }
    return min(max(id, 0), vocab - 1);
}
#endif

}  // namespace tmb
