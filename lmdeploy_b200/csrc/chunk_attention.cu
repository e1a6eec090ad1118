// Attention within chunks with sigmoid weights that are mixed across heads (ChunkAttention in mixers.h): the kernel for any
// head size and number in both element types, and the choice among the kernels.  New keys and values go into the token rings
// by the window attention's writer.
#include "chunk_attention.h"
#include "common.cuh"
#include "tm_b200.h"

#include <algorithm>

namespace tmb {
namespace {

constexpr int kMaxHeadDim = 256, kTile = 32;

// One CTA per (query, sequence), all heads.  In tiles of 32 keys: a warp takes heads in turn (lane = key), then the weights
// are mixed, then every thread adds to its own elements of the output, which live in shared memory.
template<typename E>
__global__ void __launch_bounds__(512) chunk_attention_kernel(const ChunkKernelParams p)
{
    extern __shared__ __align__(16) float sm[];
    pdl_wait();
    pdl_launch_dependents();
    const ChunkAttention& a = p.a;
    const SeqSpan         s = p.c.spans[blockIdx.y];
    if ((int)blockIdx.x >= s.n || !s.live) return;
    const int i = s.history + blockIdx.x, t = s.tok0 + blockIdx.x, H = a.heads, group = H / a.kv_heads;
    float *   q = sm, *o = q + H * a.dim, *w = o + H * a.vdim, *m = w + H * kTile;
    const int threads = blockDim.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const E*  row = static_cast<const E*>(p.c.proj) + (size_t)t * p.c.proj_ld + a.q_col;
    for (int d = threadIdx.x; d < H * a.dim; d += threads) q[d] = to_f32(row[d]);
    for (int d = threadIdx.x; d < H * a.vdim; d += threads) o[d] = 0.f;
    const E*  keys = reinterpret_cast<const E*>(s.slab + a.k_off);
    const E*  vals = reinterpret_cast<const E*>(s.slab + a.v_off);
    const int first = chunk_first(i, a.chunk);
    __syncthreads();
    for (int j0 = first; j0 <= i; j0 += kTile) {
        const int n = min(kTile, i + 1 - j0);
        for (int g = warp; g < H; g += threads / 32) {
            float x = 0.f;
            if (lane < n) {
                const E*     k  = keys + ((size_t)(g / group) * a.ring + (j0 + lane) % a.ring) * a.dim;
                const float* qg = q + g * a.dim;
                float        s4[4] = {};
                int          d = 0;
                for (; d + 4 <= a.dim; d += 4) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) s4[e] = fmaf(to_f32(k[d + e]), qg[d + e], s4[e]);
                }
                for (; d < a.dim; ++d) s4[0] = fmaf(to_f32(k[d]), qg[d], s4[0]);
                x = sigmoid_f32(((s4[0] + s4[1]) + (s4[2] + s4[3])) * a.scale + a.bias[g]);
            }
            w[g * kTile + lane] = x;
        }
        __syncthreads();
        for (int e = threadIdx.x; e < H * kTile; e += threads) {
            const int h = e / kTile, j = e % kTile;
            float     x = 0.f;
            for (int g = 0; g < H; ++g) x = fmaf(a.talk[h * H + g], w[g * kTile + j], x);
            m[e] = x;
        }
        __syncthreads();
        for (int e = threadIdx.x; e < H * a.vdim; e += threads) {
            const int h = e / a.vdim, d = e - h * a.vdim;
            const E*  v = vals + (size_t)(h / group) * a.ring * a.vdim + d;
            float     x = o[e];
            for (int j = 0; j < n; ++j) x = fmaf(m[h * kTile + j], to_f32(v[(size_t)((j0 + j) % a.ring) * a.vdim]), x);
            o[e] = x;
        }
        // the next tile's weights are mixed behind its first barrier, when everybody is through with m
    }
    __syncthreads();
    E* out = static_cast<E*>(p.c.out) + (size_t)t * p.c.out_ld;
    for (int d = threadIdx.x; d < H * a.vdim; d += threads) out[d] = from_f32<E>(o[d]);
    for (int d = H * a.vdim + threadIdx.x; d < p.c.out_pad; d += threads) out[d] = from_f32<E>(0.f);
}

size_t generic_smem(const ChunkAttention& a)
{
    return (size_t)a.heads * (a.dim + a.vdim + 2 * kTile) * 4;
}

bool valid(const tm_handle* h, const ChunkAttention& a, const MixerCall& c)
{
    return a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.dim <= kMaxHeadDim && a.vdim > 0 && a.vdim <= kMaxHeadDim
           && a.chunk >= 0 && a.ring > 0 && a.bias && a.talk && c.batch > 0 && c.batch <= 65535 && c.max_n > 0
           && generic_smem(a) <= (size_t)h->max_smem;
}

int write_rows(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st)
{
    if (!a.writes) return TM_OK;
    WindowAttention w;
    w.heads = a.heads, w.kv_heads = a.kv_heads, w.dim = a.dim, w.vdim = a.vdim, w.ring = a.ring, w.k_off = a.k_off, w.v_off = a.v_off;
    w.q_col = a.q_col, w.k_col = a.k_col, w.v_col = a.v_col;
    return window_attention_write(h, w, c, st);
}

int attend(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st)
{
    const ChunkKernelParams p{a, c};
    const cudaError_t e = launch_kernel(c.f32 ? chunk_attention_kernel<float> : chunk_attention_kernel<__nv_bfloat16>, dim3(c.max_n, c.batch), dim3(512),
                                        generic_smem(a), st, c.pdl, p);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    ++h->launches;
    return TM_OK;
}

cudaError_t prepare(int max_smem)
{
    cudaError_t e = cudaFuncSetAttribute(chunk_attention_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(chunk_attention_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem);
    return e;
}
const KernelPreparation g_prepare(prepare);

}  // namespace

int chunk_attention_prefill(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st)
{
    if (!valid(h, a, c)) return TM_ERR_UNSUPPORTED;
    const int rc = write_rows(h, a, c, st);
    if (rc != TM_OK) return rc;
    if (chunk_attention_tc_supported(a, c)) return chunk_attention_tc(h, a, c, st);
    return attend(h, a, c, st);
}

int chunk_attention_decode(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st)
{
    if (!valid(h, a, c)) return TM_ERR_UNSUPPORTED;
    if (chunk_attention_step_supported(h, a, c)) return chunk_attention_step(h, a, c, st);
    const int rc = write_rows(h, a, c, st);
    return rc == TM_OK ? attend(h, a, c, st) : rc;
}

}  // namespace tmb
