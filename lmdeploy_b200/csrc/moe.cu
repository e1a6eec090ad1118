// Mixture of experts (moe.h): routing, rows to experts, and the row kernel between two layers.
#include "moe.h"
#include "common.cuh"
#include "numeric.cuh"
#include "tm_b200.h"

#include <algorithm>

namespace tmb {
namespace {

constexpr int kRouteWarps  = 8;
constexpr int kSmallTokens = 8;   // up to here every CTA routes all tokens itself: one launch instead of two

struct DispatchParams {
    MoeRouter    r;
    MoeRows      m;
    const float* logits;
    int          logits_ld;
    const void*  input;
    int          tokens, width;
};

__device__ __forceinline__ void warp_argmax(float& v, int& i)
{
#pragma unroll
    for (int m = 16; m >= 1; m >>= 1) {
        const float v2 = __shfl_xor_sync(0xffffffffu, v, m);
        const int   i2 = __shfl_xor_sync(0xffffffffu, i, m);
        if (v2 > v || (v2 == v && i2 < i)) v = v2, i = i2;
    }
}

// One warp, one token.  choice: shared, [outputs] (+ [groups] behind it); pick(k, index, weight) is called by lane 0.
template<typename Pick>
__device__ __forceinline__ void route_token(const MoeRouter& r, const float* z, float* choice, Pick pick)
{
    const int lane = threadIdx.x & 31, n = r.experts + r.identity;
    float     mx = -INFINITY, sum = 0.f;
    for (int e = lane; e < n; e += 32) mx = fmaxf(mx, z[e]);
#pragma unroll
    for (int m = 16; m >= 1; m >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, m));
    for (int e = lane; e < n; e += 32) sum += expf(z[e] - mx);
    sum = warp_sum(sum);
    for (int e = lane; e < n; e += 32) choice[e] = expf(z[e] - mx) / sum + r.correction[e];
    __syncwarp();
    if (r.keep < r.groups) {
        float*    best = choice + n;
        const int size = n / r.groups;
        for (int g = lane; g < r.groups; g += 32) {
            float b = -INFINITY;
            for (int i = 0; i < size; ++i) b = fmaxf(b, choice[g * size + i]);
            best[g] = b;
        }
        __syncwarp();
        // kept groups are marked by +infinity
        for (int k = 0; k < r.keep; ++k) {
            float v = -INFINITY;
            int   i = 1 << 30;
            for (int g = lane; g < r.groups; g += 32) {
                if (best[g] != INFINITY && (best[g] > v || i == 1 << 30)) v = best[g], i = g;
            }
            warp_argmax(v, i);
            __syncwarp();
            if (lane == 0 && i < r.groups) best[i] = INFINITY;
            __syncwarp();
        }
        for (int e = lane; e < n; e += 32) {
            if (best[e / size] != INFINITY) choice[e] = -INFINITY;
        }
        __syncwarp();
    }
    for (int k = 0; k < r.top; ++k) {
        float v = -INFINITY;
        int   i = 1 << 30;
        for (int e = lane; e < n; e += 32) {
            if (choice[e] > v) v = choice[e], i = e;
        }
        warp_argmax(v, i);
        i = min(i, n - 1);  // router outputs that are not numbers choose something, not nothing
        __syncwarp();
        if (lane == 0) {
            choice[i] = -INFINITY;
            pick(k, i, expf(z[i] - mx) / sum);
        }
        __syncwarp();
    }
}

template<typename E>
__device__ __forceinline__ void copy_row(E* dst, const E* src, int ld)
{
    // rows are multiples of 8 elements, 16-byte aligned
    constexpr int per = 16 / (int)sizeof(E);
    for (int i = threadIdx.x; i < ld / per; i += blockDim.x) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
}

// many tokens: warp per token
__global__ void __launch_bounds__(kRouteWarps * 32) moe_route_kernel(const DispatchParams p)
{
    extern __shared__ float choice[];
    pdl_wait();
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, t = blockIdx.x * kRouteWarps + warp;
    if (t >= p.tokens) return;
    route_token(p.r, p.logits + (size_t)t * p.logits_ld, choice + warp * (p.r.outputs() + p.r.groups), [&](int k, int e, float w) {
        const size_t at   = (size_t)t * p.r.top + k;
        p.m.weights[at]   = w;
        p.m.slots[at]     = e < p.r.experts ? e : -1;
        p.m.ranks[at]     = e < p.r.experts ? atomicAdd(p.m.counts + e, 1) : 0;
    });
}

// first[e] = sum of counts before e; one warp
__device__ __forceinline__ void prefix(const int* counts, int n, int* first)
{
    const int lane = threadIdx.x & 31;
    int       sum  = 0;
    for (int e0 = 0; e0 < n; e0 += 32) {
        const int own = e0 + lane < n ? counts[e0 + lane] : 0;
        int       x   = own;
#pragma unroll
        for (int m = 1; m < 32; m *= 2) {
            const int y = __shfl_up_sync(0xffffffffu, x, m);
            if (lane >= m) x += y;
        }
        if (e0 + lane < n) first[e0 + lane] = sum + x - own;
        sum += __shfl_sync(0xffffffffu, x, 31);
    }
    if (lane == 0) first[n] = sum;
}

// ... and a CTA per token that moves its row
template<typename E>
__global__ void __launch_bounds__(256) moe_gather_kernel(const DispatchParams p)
{
    extern __shared__ float dyn[];
    int* first = reinterpret_cast<int*>(dyn);
    __shared__ int slot[kMaxRouterTop];
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    if (threadIdx.x < 32) prefix(p.m.counts, p.r.experts, first);
    __syncthreads();
    if (t == 0) {
        for (int e = threadIdx.x; e <= p.r.experts; e += 256) p.m.offsets[e] = first[e];
    }
    if ((int)threadIdx.x < p.r.top) {
        const size_t at = (size_t)t * p.r.top + threadIdx.x;
        const int    e  = p.m.slots[at];
        slot[threadIdx.x] = e < 0 ? -1 : first[e] + p.m.ranks[at];
        p.m.slots[at]     = slot[threadIdx.x];
    }
    __syncthreads();
    const E* src = static_cast<const E*>(p.input) + (size_t)t * p.m.ld;
    for (int k = 0; k < p.r.top; ++k) {
        if (slot[k] >= 0) copy_row(static_cast<E*>(p.m.sorted) + (size_t)slot[k] * p.m.ld, src, p.m.ld);
    }
}

// few tokens: every CTA routes all of them and moves one row
template<typename E>
__global__ void __launch_bounds__(kRouteWarps * 32) moe_dispatch_kernel(const DispatchParams p)
{
    extern __shared__ float dyn[];
    const int n = p.r.outputs(), top = p.r.top, total = p.tokens * top;
    float*    choice = dyn;
    int*      ids    = reinterpret_cast<int*>(dyn + kRouteWarps * (n + p.r.groups));
    int *     counts = ids + total, *first = counts + p.r.experts;
    float*    weight = reinterpret_cast<float*>(first + p.r.experts + 1);  // of the CTA's own token
    int*      slot   = reinterpret_cast<int*>(weight + top);
    pdl_wait();
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, own = blockIdx.x;
    for (int e = threadIdx.x; e < p.r.experts; e += blockDim.x) counts[e] = 0;
    for (int t = warp; t < p.tokens; t += kRouteWarps) {
        route_token(p.r, p.logits + (size_t)t * p.logits_ld, choice + warp * (n + p.r.groups), [&](int k, int e, float w) {
            ids[t * top + k] = e;
            if (t == own) weight[k] = w;
        });
    }
    __syncthreads();
    for (int i = threadIdx.x; i < total; i += blockDim.x) {
        if (ids[i] < p.r.experts) atomicAdd(counts + ids[i], 1);
    }
    __syncthreads();
    if (warp == 0) prefix(counts, p.r.experts, first);
    __syncthreads();
    if (own == 0) {
        for (int e = threadIdx.x; e <= p.r.experts; e += blockDim.x) p.m.offsets[e] = first[e];
    }
    for (int k = warp; k < top; k += kRouteWarps) {
        // rank: how often the expert was chosen before
        const int e = ids[own * top + k], lane = threadIdx.x & 31;
        int       before = 0;
        for (int i = lane; i < own * top + k; i += 32) before += ids[i] == e;
#pragma unroll
        for (int m = 16; m >= 1; m >>= 1) before += __shfl_xor_sync(0xffffffffu, before, m);
        if (lane == 0) {
            slot[k] = e < p.r.experts ? first[e] + before : -1;
            p.m.slots[own * top + k] = slot[k], p.m.weights[own * top + k] = weight[k];
        }
    }
    __syncthreads();
    const E* src = static_cast<const E*>(p.input) + (size_t)own * p.m.ld;
    for (int k = 0; k < top; ++k) {
        if (slot[k] >= 0) copy_row(static_cast<E*>(p.m.sorted) + (size_t)slot[k] * p.m.ld, src, p.m.ld);
    }
}

// ------------------------------------------------------------------------------------------------ rows between layers
template<typename E, int V>
struct Chunk {
    float v[V];
    __device__ __forceinline__ void load(const E* p)
    {
        if constexpr (V == 4 && sizeof(E) == 2) {
            const uint2 w = *reinterpret_cast<const uint2*>(p);
            v[0] = bf16_lo(w.x), v[1] = bf16_hi(w.x), v[2] = bf16_lo(w.y), v[3] = bf16_hi(w.y);
        }
        else if constexpr (V == 4) {
            const float4 w = *reinterpret_cast<const float4*>(p);
            v[0] = w.x, v[1] = w.y, v[2] = w.z, v[3] = w.w;
        }
        else {
            v[0] = to_f32(*p);
        }
    }
    __device__ __forceinline__ void store(E* p) const
    {
        if constexpr (V == 4 && sizeof(E) == 2) {
            *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
        }
        else if constexpr (V == 4) {
            *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        }
        else {
            *p = from_f32<E>(v[0]);
        }
    }
};

template<typename E, int V>
__global__ void __launch_bounds__(512) norm_rows_kernel(const RowsCall c)
{
    extern __shared__ __align__(16) float row[];
    __shared__ float red[16];
    __shared__ int   slot[kMaxRouterTop];
    __shared__ float weight[kMaxRouterTop];
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x, W = c.width;
    float*    x = c.x + (size_t)t * W;
    if (t == 0) {
        for (int i = threadIdx.x; i < c.clear_count; i += blockDim.x) c.clear[i] = 0;
    }
    if (c.expert_rows && (int)threadIdx.x < c.top) {
        slot[threadIdx.x]   = c.slots[(size_t)t * c.top + threadIdx.x];
        weight[threadIdx.x] = c.weights[(size_t)t * c.top + threadIdx.x];
    }
    __syncthreads();
    const E* token = c.ids ? static_cast<const E*>(c.embed) + (size_t)min(max(c.ids[t], 0), c.vocab - 1) * W : nullptr;
    float    sq    = 0.f;
    for (int i = V * threadIdx.x; i < W; i += V * blockDim.x) {
        Chunk<float, V> r;
        if (token) {
            Chunk<E, V> e;
            e.load(token + i);
#pragma unroll
            for (int j = 0; j < V; ++j) r.v[j] = e.v[j];
        }
        else {
            r.load(x + i);
        }
        if (c.expert_rows) {
            Chunk<E, V>     g;
            Chunk<float, V> b;
            float           sum[V] = {};
            g.load(static_cast<const E*>(c.gate) + (size_t)t * c.gate_ld + i);
            b.load(c.gate_bias + i);
            for (int k = 0; k < c.top; ++k) {
                Chunk<E, V> y;
                y.load(slot[k] < 0 ? static_cast<const E*>(c.input) + (size_t)t * c.input_ld + i : static_cast<const E*>(c.expert_rows) + (size_t)slot[k] * W + i);
#pragma unroll
                for (int j = 0; j < V; ++j) sum[j] = fmaf(weight[k], y.v[j], sum[j]);
            }
#pragma unroll
            for (int j = 0; j < V; ++j) r.v[j] += c.mult * sigmoid_f32(g.v[j] + b.v[j]) * sum[j];
        }
        if (token || c.expert_rows) r.store(x + i);
#pragma unroll
        for (int j = 0; j < V; ++j) row[i + j] = r.v[j], sq += r.v[j] * r.v[j];
    }
    sq = warp_sum(sq);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
    __syncthreads();
    float total = 0.f;
    for (int i = 0; i < (int)blockDim.x / 32; ++i) total += red[i];
    const float inv = 1.f / sqrtf(total / (float)W + c.eps);
    auto put = [&](void* out, const float* weights) {
        E* dst = static_cast<E*>(out) + (size_t)t * c.out_ld;
        for (int i = V * threadIdx.x; i < W; i += V * blockDim.x) {
            Chunk<float, V> w;
            Chunk<E, V>     y;
            w.load(weights + i);
#pragma unroll
            for (int j = 0; j < V; ++j) y.v[j] = row[i + j] * inv * w.v[j];
            y.store(dst + i);
        }
    };
    if (c.out_a) put(c.out_a, c.weight_a);
    if (c.out_b) put(c.out_b, c.weight_b);
}

template<typename E>
cudaError_t rows_launch(const RowsCall& c, cudaStream_t st, bool pdl)
{
    const int  threads = c.width >= 2048 ? 512 : (c.width >= 1024 ? 256 : 128);
    const bool quad    = c.width % 4 == 0 && c.out_ld % 4 == 0 && c.gate_ld % 4 == 0 && c.input_ld % 4 == 0 && (reinterpret_cast<uintptr_t>(c.gate) & 15) == 0;
    const auto kernel  = quad ? norm_rows_kernel<E, 4> : norm_rows_kernel<E, 1>;
    return launch_kernel(kernel, dim3(c.tokens), dim3(threads), (size_t)c.width * 4, st, pdl, c);
}

size_t small_smem(const MoeRouter& r, int tokens)
{
    return ((size_t)kRouteWarps * (r.outputs() + r.groups) + (size_t)tokens * r.top + 2 * r.experts + 1 + 2 * r.top) * 4;
}

cudaError_t prepare(int max_smem)
{
    cudaError_t e = cudaSuccess;
    auto        allow = [&](const void* f, int dynamic) {
        if (e == cudaSuccess) e = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, dynamic);
    };
    const int room = max_smem - 2048;  // beside what the kernels declare themselves
    allow((const void*)norm_rows_kernel<float, 1>, room);
    allow((const void*)norm_rows_kernel<float, 4>, room);
    allow((const void*)norm_rows_kernel<__nv_bfloat16, 1>, room);
    allow((const void*)norm_rows_kernel<__nv_bfloat16, 4>, room);
    allow((const void*)moe_route_kernel, room);
    allow((const void*)moe_dispatch_kernel<float>, room);
    allow((const void*)moe_dispatch_kernel<__nv_bfloat16>, room);
    return e;
}
const KernelPreparation g_prepare(prepare);

int finish(tm_handle* h, cudaError_t e, int launches)
{
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    h->launches += launches;
    return TM_OK;
}

}  // namespace

int moe_dispatch(tm_handle* h, const MoeRouter& r, const MoeRows& m, const float* logits, int logits_ld, const void* input, int tokens, int width,
                 bool f32, cudaStream_t st, bool pdl)
{
    const int n = r.outputs();
    if (tokens <= 0 || r.experts <= 0 || r.identity < 0 || n > kMaxRouterOutputs || r.top <= 0 || r.top > kMaxRouterTop || r.groups <= 0 || n % r.groups
        || r.keep <= 0 || r.keep > r.groups || r.top > r.keep * (n / r.groups) || m.ld % 8) {
        return TM_ERR_UNSUPPORTED;
    }
    const DispatchParams p{r, m, logits, logits_ld, input, tokens, width};
    if (tokens <= kSmallTokens) {
        const auto kernel = f32 ? moe_dispatch_kernel<float> : moe_dispatch_kernel<__nv_bfloat16>;
        return finish(h, launch_kernel(kernel, dim3(tokens), dim3(kRouteWarps * 32), small_smem(r, tokens), st, pdl, p), 1);
    }
    cudaError_t e = launch_kernel(moe_route_kernel, dim3((tokens + kRouteWarps - 1) / kRouteWarps), dim3(kRouteWarps * 32),
                                  (size_t)kRouteWarps * (n + r.groups) * 4, st, pdl, p);
    if (e != cudaSuccess) return finish(h, e, 0);
    const auto kernel = f32 ? moe_gather_kernel<float> : moe_gather_kernel<__nv_bfloat16>;
    return finish(h, launch_kernel(kernel, dim3(tokens), dim3(256), (size_t)(r.experts + 1) * 4, st, pdl, p), 2);
}

int norm_rows(tm_handle* h, const RowsCall& c, bool f32, cudaStream_t st, bool pdl)
{
    if (c.tokens <= 0 || c.width <= 0 || c.top > kMaxRouterTop || (size_t)c.width * 4 + 2048 > (size_t)h->max_smem) return TM_ERR_UNSUPPORTED;
    return finish(h, f32 ? rows_launch<float>(c, st, pdl) : rows_launch<__nv_bfloat16>(c, st, pdl), 1);
}

}  // namespace tmb
