// C ABI: per-device handles (scratch, tickets, status word, options) and what every entry point shares.
#include <mutex>
#include "handle.h"
#include "tm_b200.h"

#include <cstdlib>
#include <cstring>
#include <new>
#include <string>
#include <vector>

using namespace tmb;

namespace tmb {
thread_local int g_pdl = 0;

namespace {
std::vector<cudaError_t (*)(int)>& prepare_hooks()
{
    static std::vector<cudaError_t (*)(int)> hooks;
    return hooks;
}
}  // namespace

KernelPreparation::KernelPreparation(cudaError_t (*fn)(int))
{
    prepare_hooks().push_back(fn);
}
}  // namespace tmb

namespace {

int env_int(const char* name, int dflt)
{
    const char* v = std::getenv(name);
    return v && *v ? std::atoi(v) : dflt;
}

}  // namespace

extern "C" const char* tm_status_string(int status)
{
    switch (status) {
        case TM_OK: return "ok";
        case TM_ERR_INVALID_ARG: return "invalid argument";
        case TM_ERR_UNSUPPORTED: return "unsupported shape or option";
        case TM_ERR_WORKSPACE: return "workspace too small";
        case TM_ERR_CUDA: return "CUDA runtime error";
        case TM_ERR_DEVICE_TIMEOUT: return "a bounded device-side wait gave up";
        case TM_ERR_NCCL: return "NCCL error";
        case TM_ERR_NOT_BUILT: return "feature not built";
        case TM_ERR_IO: return "weight file missing or of the wrong size";
        default: return "unknown status";
    }
}

extern "C" int tm_create(tm_handle** out, int device)
{
    if (!out) return TM_ERR_INVALID_ARG;
    *out = nullptr;
    int prev = 0;
    if (cudaGetDevice(&prev) != cudaSuccess) return TM_ERR_CUDA;
    if (cudaSetDevice(device) != cudaSuccess) return TM_ERR_CUDA;
    tm_handle* h = new (std::nothrow) tm_handle();
    if (!h) return TM_ERR_CUDA;
    h->device = device;
    cudaDeviceProp prop{};
    cudaError_t    e = cudaGetDeviceProperties(&prop, device);
    if (e == cudaSuccess) {
        h->sm_count = prop.multiProcessorCount;
        h->max_smem = (int)prop.sharedMemPerBlockOptin;
        h->l2_bytes = prop.l2CacheSize;
        // scratch: split-K partial tiles + self-resetting tickets, status word
        // TM_B200_GEMM_SCRATCH_MB: more scratch lets one launch of the many-token GEMM cover more tokens (prefill)
        const int scratch_mb = env_int("TM_B200_GEMM_SCRATCH_MB", 256);
        h->scratch_bytes = (size_t)(scratch_mb < 64 ? 64 : (scratch_mb > 16384 ? 16384 : scratch_mb)) << 20;
        h->counter_ints  = 1u << 16;
        e                = cudaMalloc(&h->scratch, h->scratch_bytes);
    }
    if (e == cudaSuccess) e = cudaMalloc(&h->counters, h->counter_ints * sizeof(int));
    if (e == cudaSuccess) e = cudaMemset(h->counters, 0, h->counter_ints * sizeof(int));
    h->attn_scratch_bytes = 128u << 20;
    h->attn_counter_ints  = 1u << 18;
    if (e == cudaSuccess) e = cudaMalloc(&h->attn_scratch, h->attn_scratch_bytes);
    if (e == cudaSuccess) e = cudaMalloc(&h->attn_counters, h->attn_counter_ints * sizeof(int));
    if (e == cudaSuccess) e = cudaMemset(h->attn_counters, 0, h->attn_counter_ints * sizeof(int));
    if (e == cudaSuccess) e = cudaMalloc(&h->status, 256);
    if (e == cudaSuccess) e = cudaMemset(h->status, 0, 256);
    for (auto prepare : prepare_hooks()) {
        if (e == cudaSuccess) e = prepare(h->max_smem);
    }
    if (e == cudaSuccess) e = cudaDeviceSynchronize();
    h->pdl           = env_int("TM_B200_PDL", 1);
    h->p2p_allreduce = env_int("TM_B200_P2P_ALLREDUCE", 1);
    h->lm_head_cublas = env_int("TM_B200_LM_HEAD_CUBLAS", 0);
    h->fold_norm      = env_int("TM_B200_FOLD_NORM", 1);
    h->gemv_cols      = env_int("TM_B200_GEMV_COLS", 1);
    h->gemm_tc_min_n = env_int("TM_B200_GEMM_TC_MIN", 17);
    h->mmha_chunk  = env_int("TM_B200_MMHA_CHUNK", 0);
    h->mmha_warps  = env_int("TM_B200_MMHA_WARPS", 0);
    cudaSetDevice(prev);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        tm_destroy(h);
        return TM_ERR_CUDA;
    }
    *out = h;
    return TM_OK;
}

// One shared handle per device for callers that have nowhere to keep one (the header shims under include/compat, whose
// classes and free functions must keep the reference's signatures).  Created on first use, kept until the process exits.
extern "C" tm_handle* tm_handle_of_current_device(void)
{
    static std::mutex mu;
    static tm_handle* table[64] = {};
    int               dev       = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return nullptr;
    std::lock_guard<std::mutex> lock(mu);
    if (!table[dev] && tm_create(&table[dev], dev) != TM_OK) table[dev] = nullptr;
    return table[dev];
}

extern "C" int tm_destroy(tm_handle* h)
{
    if (!h) return TM_OK;
    int prev = 0;
    cudaGetDevice(&prev);
    cudaSetDevice(h->device);
    if (h->scratch) cudaFree(h->scratch);
    if (h->counters) cudaFree(h->counters);
    if (h->attn_scratch) cudaFree(h->attn_scratch);
    if (h->attn_counters) cudaFree(h->attn_counters);
    if (h->status) cudaFree(h->status);
    if (h->op_buffer) cudaFree(h->op_buffer);
    cudaSetDevice(prev);
    delete h;
    return TM_OK;
}

extern "C" int tm_last_cuda_error(const tm_handle* h)
{
    return h ? h->last_cuda_error : 0;
}

extern "C" int tm_set_option(tm_handle* h, const char* name, int value)
{
    if (!h || !name) return TM_ERR_INVALID_ARG;
    const std::string n(name);
    if (n == "gemm_tc_min_n" && value >= 1) {
        h->gemm_tc_min_n = value;
    }
    else if (n == "mmha_chunk" && value >= 0) {
        h->mmha_chunk = value;
    }
    else if (n == "mmha_warps" && (value == 0 || value == 1 || value == 2 || value == 4)) {
        h->mmha_warps = value;
    }
    else if (n == "pdl" && (value == 0 || value == 1)) {
        h->pdl = value;
    }
    else if (n == "p2p_allreduce" && (value == 0 || value == 1)) {
        // 0: the tensor-parallel decode step reduces with NCCL even where the peer-memory path is set up
        h->p2p_allreduce = value;
    }
    else if (n == "fold_norm" && (value == 0 || value == 1)) {
        h->fold_norm = value;
    }
    else if (n == "gemv_cols" && value >= 0 && value <= 2) {
        h->gemv_cols = value;
    }
    else if (n == "lm_head_cublas" && (value == 0 || value == 1)) {
        h->lm_head_cublas = value;
    }
    else if (n == "pdl_direct" && (value == 0 || value == 1)) {
        // GEMM and attention calls made DIRECTLY through this handle also launch with programmatic stream
        // serialization: the kernel may start (and request the packed weights / cache rows of earlier steps) while the
        // kernel before it in the stream still runs.  Only for callers whose preceding kernels never write those.
        h->pdl_direct = value;
    }
    else if (n == "gemm_wait_cycles" && value >= 0) {
        // bound, in SM clock cycles, of the tcgen05 GEMM's wait for the partners of a split column tile
        // (0 = the default of about a quarter of a second); tests set a tiny value to see the time-out path
        h->gemm_wait_cycles = value;
    }
    else {
        return TM_ERR_INVALID_ARG;
    }
    return TM_OK;
}

extern "C" unsigned long long tm_launch_count(const tm_handle* h)
{
    return h ? h->launches : 0ull;
}

extern "C" int tm_check_device_status(tm_handle* h, void* stream, unsigned* word)
{
    if (!h || !word) return TM_ERR_INVALID_ARG;
    cudaStream_t st = (cudaStream_t)stream;
    unsigned     w  = 0;
    cudaError_t  e  = cudaMemcpyAsync(&w, h->status, sizeof(w), cudaMemcpyDeviceToHost, st);
    if (e == cudaSuccess) e = cudaStreamSynchronize(st);
    if (e == cudaSuccess && w != 0) e = cudaMemsetAsync(h->status, 0, sizeof(unsigned), st);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    *word = w;
    return w ? TM_ERR_DEVICE_TIMEOUT : TM_OK;
}
