#include "chunk_attention.h"
#include "tm_b200.h"
namespace tmb {
bool chunk_attention_tc_supported(const ChunkAttention&, const MixerCall&) { return false; }
int  chunk_attention_tc(tm_handle*, const ChunkAttention&, const MixerCall&, cudaStream_t) { return TM_ERR_UNSUPPORTED; }
size_t chunk_attention_scratch(const ChunkAttention&, int, bool) { return 0; }
}
