// What the scheduler, the command line and the replay tool ask of a model, and the table of architectures that
// tm_model_open chooses from.  Two models implement it: the W4A16 LLaMA of llama.h and the config-driven decoder of
// decoder.h.
#pragma once

#include "handle.h"
#include "tm_b200.h"

#include <cuda_runtime.h>
#include <string>

struct tm_model {
    tm_handle* h              = nullptr;
    int        vocab_size     = 0;
    int        max_batch_size = 0;
    int        session_len    = 0;

    virtual ~tm_model() = default;
    // new tokens of some sequences through all layers; their cache / state is left one step behind the sampled token
    virtual int prefill(const tm_model_prefill_state& st, cudaStream_t s) = 0;
    // n_steps decoder steps (one token per sequence and step)
    virtual int decode(const tm_llama_decode_state& st, int n_steps, bool use_graph, cudaStream_t s) = 0;
    // a slab manager whose slabs hold what one sequence of this model caches
    virtual int new_cache(tm_cache_manager** out, size_t max_entry_count, size_t chunk_size) const = 0;
    // whether a sequence can go back to an earlier length by just forgetting cached rows (a recurrent state cannot)
    virtual bool                 can_rewind() const { return true; }
    virtual size_t               slab_bytes() const { return 0; }
    virtual unsigned long long   last_launches() const { return 0; }
};

namespace tmb {

// One entry of the table: tm_model_open takes the first whose `claims` accepts the folder.
struct ModelArchitecture {
    const char* name;
    bool (*claims)(const std::string& dir);
    int (*open)(tm_model** out, tm_handle* h, const std::string& dir, const tm_model_options& opt);
};
void register_architecture(const ModelArchitecture& a);
struct ArchitectureRegistration {
    explicit ArchitectureRegistration(const ModelArchitecture& a) { register_architecture(a); }
};

// One decode step captured into a CUDA graph, keyed by the state it was captured for.
struct StepGraph {
    cudaGraphExec_t       exec = nullptr;
    tm_llama_decode_state key{};
    unsigned long long    launches_per_step = 0;

    ~StepGraph() { drop(); }
    void drop()
    {
        if (exec) cudaGraphExecDestroy(exec);
        exec = nullptr;
    }
    // step(&launches) enqueues one step on `s`; *total = kernels launched by the call
    template<typename Step>
    int run(tm_handle* h, const tm_llama_decode_state& st, int n_steps, bool use_graph, cudaStream_t s, unsigned long long* total, Step step);
};

}  // namespace tmb

#include <cstring>

template<typename Step>
int tmb::StepGraph::run(tm_handle* h, const tm_llama_decode_state& st, int n_steps, bool use_graph, cudaStream_t s,
                        unsigned long long* total, Step step)
{
    *total = 0;
    if (!use_graph) {
        for (int i = 0; i < n_steps; ++i) {
            unsigned long long n  = 0;
            const int          rc = step(&n);
            if (rc != TM_OK) return rc;
            *total += n;
        }
        return TM_OK;
    }
    if (!exec || std::memcmp(&key, &st, sizeof(st)) != 0) {
        drop();
        if (s == nullptr) return TM_ERR_INVALID_ARG;  // the legacy stream cannot be captured
        cudaGraph_t g = nullptr;
        if (cudaStreamBeginCapture(s, cudaStreamCaptureModeThreadLocal) != cudaSuccess) return TM_ERR_CUDA;
        unsigned long long n  = 0;
        const int          rc = step(&n);
        const cudaError_t  e  = cudaStreamEndCapture(s, &g);
        if (rc != TM_OK || e != cudaSuccess || !g) {
            if (g) cudaGraphDestroy(g);
            h->last_cuda_error = (int)e;
            return rc != TM_OK ? rc : TM_ERR_CUDA;
        }
        const cudaError_t ei = cudaGraphInstantiate(&exec, g, 0);
        cudaGraphDestroy(g);
        if (ei != cudaSuccess) {
            exec               = nullptr;
            h->last_cuda_error = (int)ei;
            return TM_ERR_CUDA;
        }
        key               = st;
        launches_per_step = n;
    }
    for (int i = 0; i < n_steps; ++i) {
        if (cudaGraphLaunch(exec, s) != cudaSuccess) return TM_ERR_CUDA;
    }
    *total = launches_per_step * (unsigned long long)n_steps;
    return TM_OK;
}
