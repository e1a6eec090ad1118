// Replay of given token ids through a served model: the scheduler's two calls (tm_model_prefill for several tokens,
// tm_model_decode for one) on cache slabs of the model's own manager, with the logits handed to the host instead of a
// sampler.
#include "model.h"

#include <new>
#include <unordered_map>
#include <vector>

using namespace tmb;

struct tm_replay {
    tm_model*                                       model  = nullptr;
    tm_cache_manager*                               cache  = nullptr;
    cudaStream_t                                    stream = nullptr;
    std::unordered_map<uint64_t, tm_cache_sequence> live;  // cache_len = tokens taken in
    void **                                         d_k = nullptr, **d_v = nullptr;
    int *                                           d_len = nullptr, *d_forced = nullptr, *d_out = nullptr, *d_step = nullptr;
    float *                                         d_logits = nullptr, *d_rows = nullptr;
    size_t                                          rows_capacity = 0;
};

extern "C" int tm_replay_destroy(tm_replay* r)
{
    if (!r) return TM_OK;
    int prev = 0;
    cudaGetDevice(&prev);
    cudaSetDevice(r->model->h->device);
    if (r->stream) cudaStreamSynchronize(r->stream);
    for (void* p : {(void*)r->d_k, (void*)r->d_v, (void*)r->d_len, (void*)r->d_forced, (void*)r->d_out, (void*)r->d_step, (void*)r->d_logits,
                    (void*)r->d_rows}) {
        if (p) cudaFree(p);
    }
    if (r->cache) tm_cache_manager_destroy(r->cache);
    if (r->stream) cudaStreamDestroy(r->stream);
    cudaSetDevice(prev);
    delete r;
    return TM_OK;
}

extern "C" int tm_replay_create(tm_replay** out, tm_model* model, size_t max_sequences)
{
    if (!out || !model || !max_sequences) return TM_ERR_INVALID_ARG;
    *out         = nullptr;
    tm_replay* r = new (std::nothrow) tm_replay();
    if (!r) return TM_ERR_CUDA;
    r->model = model;
    int prev = 0;
    cudaGetDevice(&prev);
    cudaSetDevice(model->h->device);
    bool ok = cudaStreamCreateWithFlags(&r->stream, cudaStreamNonBlocking) == cudaSuccess && cudaMalloc((void**)&r->d_k, sizeof(void*)) == cudaSuccess
              && cudaMalloc((void**)&r->d_v, sizeof(void*)) == cudaSuccess && cudaMalloc((void**)&r->d_len, 4) == cudaSuccess
              && cudaMalloc((void**)&r->d_forced, 4) == cudaSuccess && cudaMalloc((void**)&r->d_out, 4) == cudaSuccess
              && cudaMalloc((void**)&r->d_step, 4) == cudaSuccess && cudaMalloc((void**)&r->d_logits, (size_t)model->vocab_size * 4) == cudaSuccess;
    const int rc = ok ? tm_model_new_cache(model, max_sequences, 1, &r->cache) : TM_ERR_CUDA;
    cudaSetDevice(prev);
    if (rc != TM_OK) {
        tm_replay_destroy(r);
        return rc;
    }
    *out = r;
    return TM_OK;
}

extern "C" int tm_replay_step(tm_replay* r, uint64_t id, const int* tokens, int count, const int* want, int want_count, float* logits)
{
    if (!r || !tokens || count <= 0 || want_count < 0 || (want_count > 0 && (!want || !logits))) return TM_ERR_INVALID_ARG;
    tm_model&    m = *r->model;
    const size_t V = (size_t)m.vocab_size;
    cudaStream_t s = r->stream;
    int          prev = 0, rc = TM_OK;
    cudaGetDevice(&prev);
    cudaSetDevice(m.h->device);
    struct Restore {
        int d;
        ~Restore() { cudaSetDevice(d); }
    } restore{prev};
    auto it = r->live.find(id);
    if (it == r->live.end()) {
        tm_cache_sequence q{};
        if ((rc = tm_cache_create(r->cache, id, s, &q)) != TM_OK) return rc;
        it = r->live.emplace(id, q).first;
    }
    tm_cache_sequence& q       = it->second;
    const int          history = (int)q.cache_len;
    if (history + count > m.session_len) return TM_ERR_WORKSPACE;
    const float* rows = nullptr;
    if (count == 1) {
        for (int i = 0; i < want_count; ++i) {
            if (want[i] != 0) return TM_ERR_INVALID_ARG;
        }
        if (cudaMemcpyAsync(r->d_k, &q.k_cache, sizeof(void*), cudaMemcpyHostToDevice, s) != cudaSuccess
            || cudaMemcpyAsync(r->d_v, &q.v_cache, sizeof(void*), cudaMemcpyHostToDevice, s) != cudaSuccess
            || cudaMemcpyAsync(r->d_len, &history, 4, cudaMemcpyHostToDevice, s) != cudaSuccess
            || cudaMemcpyAsync(r->d_forced, tokens, 4, cudaMemcpyHostToDevice, s) != cudaSuccess || cudaMemsetAsync(r->d_step, 0, 4, s) != cudaSuccess) {
            return TM_ERR_CUDA;
        }
        tm_llama_decode_state st{};
        st.batch_size = 1, st.max_steps = 1, st.k_cache_ptrs = r->d_k, st.v_cache_ptrs = r->d_v, st.sequence_lengths = r->d_len;
        st.forced_ids = r->d_forced, st.output_ids = r->d_out, st.step = r->d_step, st.logits_out = r->d_logits;
        rc   = tm_model_decode(&m, &st, 1, 1, s);
        rows = r->d_logits;
    }
    else {
        if ((size_t)want_count > r->rows_capacity) {
            if (r->d_rows) cudaFree(r->d_rows);
            r->d_rows = nullptr, r->rows_capacity = 0;
            if (cudaMalloc((void**)&r->d_rows, want_count * V * 4) != cudaSuccess) return TM_ERR_CUDA;
            r->rows_capacity = want_count;
        }
        const int              cu[2] = {0, count};
        tm_model_prefill_state st{};
        st.batch_size = 1, st.input_ids = tokens, st.cu_seqlens = cu, st.history_lengths = &history, st.k_cache = &q.k_cache, st.v_cache = &q.v_cache;
        st.want_count = want_count, st.want = want, st.logits_out = r->d_rows;
        rc   = tm_model_prefill(&m, &st, s);
        rows = r->d_rows;
    }
    if (rc != TM_OK) return rc;
    q.cache_len += count;
    for (int i = 0; i < (count == 1 ? want_count : 1); ++i) {
        const size_t n = count == 1 ? V : want_count * V;
        if (want_count > 0 && cudaMemcpyAsync(logits + i * V, rows, n * 4, cudaMemcpyDeviceToHost, s) != cudaSuccess) return TM_ERR_CUDA;
    }
    unsigned word = 0;
    return tm_model_check_status(&m, s, &word);  // synchronises
}

extern "C" int tm_replay_end(tm_replay* r, uint64_t id)
{
    if (!r || !r->live.count(id)) return TM_ERR_INVALID_ARG;
    r->live.erase(id);
    return tm_cache_erase(r->cache, id);
}
