#include "chunk_attention.h"
#include "tm_b200.h"
namespace tmb {
bool chunk_attention_step_supported(const tm_handle*, const ChunkAttention&, const MixerCall&) { return false; }
int  chunk_attention_step(tm_handle*, const ChunkAttention&, const MixerCall&, cudaStream_t) { return TM_ERR_UNSUPPORTED; }
}
