// The served-model interface of the C ABI: architecture table, open / close, prefill, decode, cache.
#include "model.h"

#include <vector>

using namespace tmb;

namespace {

std::vector<ModelArchitecture>& architectures()
{
    static std::vector<ModelArchitecture> table;
    return table;
}

}  // namespace

namespace tmb {
void register_architecture(const ModelArchitecture& a)
{
    architectures().push_back(a);
}
}  // namespace tmb

extern "C" int tm_model_open(tm_model** out, tm_handle* h, const char* dir, const tm_model_options* opt)
{
    if (!out || !h || !dir || !opt || opt->max_batch_size <= 0 || opt->session_len <= 1 || opt->max_prefill_tokens < 0) {
        return TM_ERR_INVALID_ARG;
    }
    if (opt->dtype != TM_DTYPE_BF16 && opt->dtype != TM_DTYPE_F32) return TM_ERR_INVALID_ARG;
    *out = nullptr;
    for (const ModelArchitecture& a : architectures()) {
        if (a.claims(dir)) return a.open(out, h, dir, *opt);
    }
    return TM_ERR_UNSUPPORTED;
}

extern "C" int tm_model_close(tm_model* m)
{
    if (!m) return TM_OK;
    int prev = 0;
    cudaGetDevice(&prev);
    cudaSetDevice(m->h->device);
    delete m;
    cudaSetDevice(prev);
    return TM_OK;
}

extern "C" int tm_model_architectures(char* names, size_t capacity)
{
    std::string all;
    for (const ModelArchitecture& a : architectures()) all += (all.empty() ? "" : ",") + std::string(a.name);
    if (!names || capacity < all.size() + 1) return TM_ERR_WORKSPACE;
    std::memcpy(names, all.c_str(), all.size() + 1);
    return TM_OK;
}

extern "C" int tm_model_describe(const tm_model* m, tm_model_info* info)
{
    if (!m || !info) return TM_ERR_INVALID_ARG;
    info->vocab_size     = m->vocab_size;
    info->max_batch_size = m->max_batch_size;
    info->session_len    = m->session_len;
    info->can_rewind     = m->can_rewind() ? 1 : 0;
    info->slab_bytes     = m->slab_bytes();
    return TM_OK;
}

extern "C" int tm_model_new_cache(const tm_model* m, size_t max_entry_count, size_t chunk_size, tm_cache_manager** out)
{
    if (!m || !out || !max_entry_count || !chunk_size) return TM_ERR_INVALID_ARG;
    return m->new_cache(out, max_entry_count, chunk_size);
}

extern "C" int tm_model_prefill(tm_model* m, const tm_model_prefill_state* st, void* stream)
{
    if (!m || !st || st->batch_size < 0 || st->want_count < 0) return TM_ERR_INVALID_ARG;
    if (st->batch_size == 0) return TM_OK;
    if (!st->input_ids || !st->cu_seqlens || !st->history_lengths || !st->k_cache || !st->v_cache) return TM_ERR_INVALID_ARG;
    if (st->want_count > 0 && (!st->want || !st->logits_out)) return TM_ERR_INVALID_ARG;
    const int total = st->cu_seqlens[st->batch_size];
    if (st->cu_seqlens[0] != 0) return TM_ERR_INVALID_ARG;
    for (int b = 0; b < st->batch_size; ++b) {
        const int n = st->cu_seqlens[b + 1] - st->cu_seqlens[b];
        if (n < 0 || st->history_lengths[b] < 0 || st->history_lengths[b] + n > m->session_len || !st->k_cache[b]) return TM_ERR_INVALID_ARG;
    }
    for (int i = 0; i < total; ++i) {
        if (st->input_ids[i] < 0 || st->input_ids[i] >= m->vocab_size) return TM_ERR_INVALID_ARG;
    }
    for (int i = 0; i < st->want_count; ++i) {
        if (st->want[i] < 0 || st->want[i] >= total || (i > 0 && st->want[i] <= st->want[i - 1])) return TM_ERR_INVALID_ARG;
    }
    int prev = 0;
    cudaGetDevice(&prev);
    cudaSetDevice(m->h->device);
    const int rc = m->prefill(*st, (cudaStream_t)stream);
    cudaSetDevice(prev);
    return rc;
}

extern "C" int tm_model_decode(tm_model* m, const tm_llama_decode_state* st, int n_steps, int use_graph, void* stream)
{
    if (!m || !st || n_steps < 0) return TM_ERR_INVALID_ARG;
    if (st->batch_size <= 0 || st->batch_size > m->max_batch_size || st->max_steps <= 0) return TM_ERR_INVALID_ARG;
    if (!st->k_cache_ptrs || !st->v_cache_ptrs || !st->sequence_lengths || !st->output_ids || !st->step) return TM_ERR_INVALID_ARG;
    return m->decode(*st, n_steps, use_graph != 0, (cudaStream_t)stream);
}

extern "C" unsigned long long tm_model_last_launches(const tm_model* m)
{
    return m ? m->last_launches() : 0ull;
}

extern "C" int tm_model_check_status(tm_model* m, void* stream, unsigned* word)
{
    if (!m) return TM_ERR_INVALID_ARG;
    return tm_check_device_status(m->h, stream, word);
}
