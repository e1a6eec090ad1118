// Config-driven decoder: a model whose layer list, mixers and sizes come from config.json.  Each layer is parallel.
//
// LayerForm::kScalarNorm: x <- x + mixer(h) + ff(h) with h = norm(x), which makes it two GEMMs around a mixer:
//   input GEMM    all projections of the mixer and the gated pair of the feed-forward, stacked in one weight; the norm is
//                 one number per token (its gain is one number), so it scales the rows of the product
//   mixer         window attention or delta rule (mixers.h), from and to the same buffers
//   output GEMM   [mixer's output weight | feed-forward's down weight] over the concatenated inputs, added to the residual
//
// LayerForm::kGatedBranches: x <- x + m (sigmoid(A1 h1 + b1) mixer(h1) + sigmoid(A2 h2 + b2) experts(h2)), h1 and h2 two
// norms of x with weight vectors:
//   rows kernel   what the experts of the layer ahead add to x, then h1 and h2 (moe.h)
//   input GEMM    [mixer's projections | A1] over h1 and [A2 | router, in fp32] over h2 in one launch
//   mixer, output GEMM   its epilogue adds the gated product to the residual
//   experts       dispatch, then the (gate, up) pairs and the down projections as two grouped GEMMs
//
// Slab of a sequence: per attention layer the token rings of keys and values and the pooled rows, per recurrent layer the
// fp32 state, each on a 256-byte boundary.
#pragma once
#include "gemm_dense.h"
#include "json.h"
#include "mixers.h"
#include "moe.h"
#include "model.h"

#include <string>
#include <vector>

namespace tmb {

enum class MixerType : int { kAttention, kGeneralDelta, kChunkAttention, kGatedLinear };
enum class LayerForm : int { kScalarNorm, kGatedBranches };

struct MixerSpec {
    MixerType type  = MixerType::kAttention;
    int       heads = 0, dim = 0;
    // attention
    int    kv_heads = 0, vdim = 0;
    int    rot_dims = 0;
    double rot_base = 10000.0, rot_factor = 1.0;
    double scale = 1.0, softcap = 0.0;
    int    window = 0, pool = 0;
    // chunk attention: tokens of a chunk (0: one chunk), the layer whose keys and values it uses (-1: its own)
    int chunk = 0, kv_from = -1;
    // general delta, gated linear: rank of the decay's low-rank projection (given by the shape of its tensors)
    int rank = 0;
    // gated linear
    double tau = 1.0;

    int out_width() const { return heads * (type == MixerType::kGeneralDelta ? dim : vdim); }
};

struct MoeSpec {
    int    experts = 0, identity = 0, top = 0, groups = 1, keep = 1;  // as in MoeRouter; experts 0: no mixture
    int    ff    = 0;
    double limit = 0;
};

struct LayerSpec {
    MixerSpec mixer;
    int       ff = 0;  // dense feed-forward, 0: none
    MoeSpec   moe;
};

struct DecoderConfig {
    std::string            architecture;
    int                    vocab = 0, width = 0;
    LayerForm              form = LayerForm::kScalarNorm;
    double                 norm_eps = 0, embedding_scale = 1.0, residual_mult = 1.0;
    std::vector<LayerSpec> layers;
};

// config.json of one of the architectures -> DecoderConfig; false with a reason when something is missing or impossible
bool read_decoder_config(const Json& j, DecoderConfig* c, std::string* why);

constexpr float kSwishSlope = 1.702f;  // of the clamped experts

struct DecoderLayer {
    LayerSpec       spec;
    WindowAttention attention;
    DeltaRule       delta;
    ChunkAttention  chunk;
    GatedLinear     linear;
    int             mixer_cols = 0;  // projection columns, a multiple of kDenseTile
    int             in_rows    = 0;  // mixer_cols + 2 ff, rounded up to kDenseTile
    int             mix_pad    = 0;  // columns of the output GEMM's input that belong to the mixer
    int             out_k      = 0;  // all columns of it
    int             tanh_lo = 0, tanh_hi = 0;
    void *          w_in = nullptr, *w_out = nullptr, *w2 = nullptr;  // element type
    float *         gain = nullptr, *w0 = nullptr, *a_bias = nullptr, *norm = nullptr, *inv_freq = nullptr;
    // gated branches
    MoeRouter router;
    int       x2_from = 0, rg1_col = 0, rg2_col = 0, router_col = 0;  // columns of the input GEMM; x2_from 0: no feed-forward
    float *   norm1 = nullptr, *norm2 = nullptr, *rg1_bias = nullptr, *rg2_bias = nullptr, *correction = nullptr;
    void *    w_experts = nullptr, *w_down = nullptr;  // [expert][2 ff][width], [expert][width][ff]
    float *   bias = nullptr, *talk = nullptr;
    void*     talk_half = nullptr;
};

// Where a checkpoint tensor goes: rows x cols at `dst`, row r at dst + r * row_stride (elements)
struct WeightTarget {
    std::string name;
    int64_t     rows = 0, cols = 0;
    bool        scalar = false, vector = false;  // shape [] / [cols]
    void*       dst = nullptr;
    int64_t     row_stride = 0;
    bool        f32 = false;      // kept in fp32 whatever the element type
    float       init_std = 0.f, init_mean = 0.f;  // random initialisation
};

}  // namespace tmb

struct tm_decoder final : tm_model {
    tmb::DecoderConfig             cfg;
    bool                           f32 = false;
    int                            max_prefill = 0;  // tokens of one pass through the layers
    std::vector<tmb::DecoderLayer> layers;
    std::vector<tmb::WeightTarget> targets;
    size_t                         slab = 0;
    int                            x_ld = 0, proj_ld = 0, y_ld = 0;

    std::vector<void*> owned;
    void *             embed = nullptr, *head = nullptr;
    float*             final_gain = nullptr;
    // activations of one pass
    float *       x = nullptr, *ssq = nullptr, *delta_scratch = nullptr, *logits = nullptr;
    void *        xb = nullptr, *proj = nullptr, *y = nullptr, *want_xb = nullptr;
    float*        want_ssq = nullptr;
    int           ssq_stride = 0;
    // gated branches: second norm, router logits, rows of the experts
    void *        xb2 = nullptr, *expert_act = nullptr, *expert_out = nullptr, *attention_weights = nullptr;
    float *       router_logits = nullptr, *final_norm = nullptr;
    int           router_ld = 0, act_ld = 0;
    size_t        attention_weights_bytes = 0;
    tmb::MoeRows  moe_rows;
    tmb::QueryTile* tiles = nullptr;
    int *         ids = nullptr, *want = nullptr, *picked = nullptr;
    unsigned char* inactive = nullptr;
    tmb::SeqSpan* spans = nullptr;
    tmb::StepGraph graph;
    unsigned long long launches_of_last = 0;

    ~tm_decoder() override;
    int    init(tm_handle* handle, const tmb::DecoderConfig& c, const tm_model_options& opt);
    int    load(const std::string& safetensors, std::string* why);
    int    random_weights(unsigned long long seed);
    int    prefill(const tm_model_prefill_state& st, cudaStream_t s) override;
    int    decode(const tm_llama_decode_state& st, int n_steps, bool use_graph, cudaStream_t s) override;
    int    new_cache(tm_cache_manager** out, size_t max_entry_count, size_t chunk_size) const override;
    bool   can_rewind() const override { return false; }
    size_t slab_bytes() const override { return slab; }
    unsigned long long last_launches() const override { return launches_of_last; }

private:
    struct Pass;
    int  run_layers(const Pass& p, cudaStream_t s);
    int  run_gated_layers(const Pass& p, cudaStream_t s);
    int  run_mixer(const tmb::DecoderLayer& L, const Pass& p, cudaStream_t s);
    int  copy_residual(const Pass& p, size_t layer, cudaStream_t s);
    int  derive_weights();
    int  step(const tm_llama_decode_state& st, cudaStream_t s, unsigned long long* launches);
    bool alloc(void** p, size_t bytes);
};
