// Sequence mixers of the config-driven decoder: softmax attention over a sliding window with pooled blocks behind it,
// attention within chunks with sigmoid weights mixed across heads, a recurrence with a generalised delta rule, and gated
// linear attention.  Every size and constant is a field; sequences are described by spans.
#pragma once
#include "handle.h"

#include <cuda_runtime.h>

namespace tmb {

// The new tokens of one sequence in a launch: rows [tok0, tok0 + n) of the activations, positions history, history + 1, ...
struct SeqSpan {
    unsigned char* slab    = nullptr;  // what the sequence caches (layout: decoder.h)
    int            history = 0;
    int            n       = 0;
    int            tok0    = 0;
    int            live    = 0;        // 0: the sequence sits this step out and nothing of it is written
};

struct WindowAttention {
    int          heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    int          rot_dims = 0;           // leading dimensions that rotate, pairs (2i, 2i + 1)
    const float* inv_freq = nullptr;     // device [rot_dims / 2]
    float        scale = 1.f, softcap = 0.f;  // softcap 0: none
    // A position i sees the tokens j with 0 <= i - j < window (0: all), and the mean key / value of every block of `pool`
    // tokens (0: none) that ends at or before i - window.
    int          window = 0, pool = 0;
    // Token rows live in a ring: position p in row p % ring.  A ring holds the window (and a block) of the oldest query
    // of a launch and all tokens of the launch.  Pooled rows: one per block.
    int          ring = 0, pool_rows = 0;
    size_t       k_off = 0, v_off = 0, pk_off = 0, pv_off = 0;  // bytes in the slab; [kv head][row][dim or vdim]
    int          q_col = 0, k_col = 0, v_col = 0, g_col = 0;    // columns of the projections; g: one gate logit per head
};

// 128 consecutive query tokens of one span (the last tile of a span may be shorter)
struct QueryTile {
    int span = 0, q0 = 0;
};

// proj [tokens][proj_ld] (q is rotated in place in prefill), out [tokens][out_ld]: columns [0, heads * vdim) get the gated
// output, [heads * vdim, out_pad) zeros.  spans: device array.  max_n: the longest span; max_context: upper bound on
// history + n.
struct MixerCall {
    void*          proj     = nullptr;
    int            proj_ld  = 0;
    void*          out      = nullptr;
    int            out_ld   = 0, out_pad = 0;
    const SeqSpan* spans    = nullptr;
    int            batch    = 0, tokens = 0, max_n = 0, max_context = 0;
    bool           f32      = false;
    bool           pdl      = false;
    const QueryTile* tiles  = nullptr;  // device, prefill: the query tiles of all spans in turn (null: unknown)
    int            tile_count = 0;
};
int window_attention_prefill(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st);
int window_attention_decode(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st);

// The new keys and values of the spans into the token rings, rotated if rot_dims says so (the first step of the attention
// calls; q is rotated in place).
int window_attention_write(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st);

// Attention without a softmax: position i sees the tokens from the start of its chunk (positions counted from the start of
// the sequence) to itself; head g gives key j the weight sigmoid(scale q.k + bias[g]), and head h applies
// sum_g talk[h][g] weight_g to its own values.  No positions in the scores.
struct ChunkAttention {
    int          heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float        scale = 1.f;
    int          chunk = 0;             // tokens of a chunk, 0: one chunk
    const float* bias  = nullptr;       // [heads]
    const float* talk  = nullptr;       // [heads][heads]
    const void*  talk_half = nullptr;   // fp16 [talk_pad(heads)][talk_pad(heads)], zeros beyond the heads
    bool         writes = true;         // false: keys and values are another layer's, which ran before
    int          ring = 0;              // as in WindowAttention
    size_t       k_off = 0, v_off = 0;
    int          q_col = 0, k_col = 0, v_col = 0;
    void*        weights = nullptr;     // scratch of a prefill
    size_t       weights_bytes = 0;
};
constexpr int talk_pad(int heads)
{
    return (heads + 15) / 16 * 16;
}
// scratch that lets a prefill run on the tensor core with at least one query tile at a time; 0: it runs without
size_t chunk_attention_scratch(const ChunkAttention& a, int max_context, bool f32);
int    chunk_attention_prefill(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st);
int    chunk_attention_decode(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st);

struct DeltaRule {
    int          heads = 0, dim = 0;
    int          rank     = 0;         // of the decay's low-rank projection
    const void*  w2       = nullptr;   // [heads * dim][w2_ld], element type
    int          w2_ld    = 0;
    const float* w0       = nullptr;   // [heads * dim]
    const float* a_bias   = nullptr;   // [heads * dim]
    const float* norm     = nullptr;   // [heads * dim], weight behind the per-head norm
    float        norm_eps = 0.f;
    float        unit_eps = 1e-6f;     // u = k / sqrt(sum k^2 + unit_eps)
    float        decay_scale = 0.60653065971263342f;  // decay = exp(-decay_scale * sigmoid(.)); here exp(-1/2)
    size_t       state_off = 0;        // bytes in the slab: float [head][value dim][key dim]
    int          r_col = 0, k_col = 0, v_col = 0, a_col = 0, g_col = 0, w1_col = 0;  // columns of the projections; w1 after tanh
};
// scratch of a prefill, fp32: so many floats per token
size_t delta_rule_scratch_floats(const DeltaRule& d);
int    delta_rule_prefill(tm_handle* h, const DeltaRule& d, const MixerCall& c, float* scratch, cudaStream_t st);
int delta_rule_decode(tm_handle* h, const DeltaRule& d, const MixerCall& c, cudaStream_t st);

// Gated linear attention, per head: S <- diag(decay) S + k v^T, o = S^T (scale q), decay = sigmoid(w2 a + bias)^(1/tau) per
// key channel with a the low-rank projection; then o over its root mean square times `norm`, times silu of the gate.
struct GatedLinear {
    int          heads = 0, dim = 0, vdim = 0;
    int          rank     = 0;
    const void*  w2       = nullptr;  // [heads * dim][w2_ld], element type
    int          w2_ld    = 0;
    const float* bias     = nullptr;  // [heads * dim]
    const float* norm     = nullptr;  // [vdim]
    float        norm_eps = 0.f, scale = 1.f, tau = 1.f;
    size_t       state_off = 0;       // bytes in the slab: float [head][value channel][key channel]
    int          q_col = 0, k_col = 0, v_col = 0, g_col = 0, a_col = 0;
};
size_t gated_linear_scratch_floats(const GatedLinear& d);  // of a prefill, per token
int    gated_linear_prefill(tm_handle* h, const GatedLinear& d, const MixerCall& c, float* scratch, cudaStream_t st);
int    gated_linear_decode(tm_handle* h, const GatedLinear& d, const MixerCall& c, cudaStream_t st);

}  // namespace tmb
