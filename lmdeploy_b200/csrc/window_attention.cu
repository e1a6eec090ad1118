// Softmax attention over a sliding window, with the tokens that have left it pooled in blocks (WindowAttention in
// mixers.h): cache writers, and attention kernels for any head size in both element types.  Head sizes the tensor core
// takes have kernels of their own (window_attention_tc.cu, window_attention_decode.cu).
#include "common.cuh"
#include "window_attention.h"
#include "tm_b200.h"

namespace tmb {
namespace {

constexpr int kMaxHeadDim = 256;

template<typename E>
__device__ __forceinline__ E* slab_rows(unsigned char* slab, size_t off)
{
    return reinterpret_cast<E*>(slab + off);
}

// One CTA per new token: q rotated in place, k rotated and v copied into the token ring.
template<typename E>
__global__ void __launch_bounds__(128) window_write_kernel(const WindowKernelParams p)
{
    __shared__ float cs[kMaxHeadDim / 2], sn[kMaxHeadDim / 2];
    pdl_wait();
    pdl_launch_dependents();
    const WindowAttention& a = p.a;
    const SeqSpan          s = p.c.spans[blockIdx.y];
    if ((int)blockIdx.x >= s.n || !s.live) return;
    const int pos = s.history + blockIdx.x;
    E*        row = static_cast<E*>(p.c.proj) + (size_t)(s.tok0 + blockIdx.x) * p.c.proj_ld;
    for (int i = threadIdx.x; i < a.rot_dims / 2; i += blockDim.x) sincosf((float)pos * a.inv_freq[i], &sn[i], &cs[i]);
    __syncthreads();
    const int slot = pos % a.ring;
    const int half = (a.dim + 1) / 2;
    for (int w = threadIdx.x; w < (a.heads + a.kv_heads) * half; w += blockDim.x) {
        const int  hh = w / half, i = w - hh * half, d = 2 * i;
        const bool is_q = hh < a.heads;
        E*         src  = row + (is_q ? a.q_col + hh * a.dim : a.k_col + (hh - a.heads) * a.dim) + d;
        E*         dst  = is_q ? src : slab_rows<E>(s.slab, a.k_off) + ((size_t)(hh - a.heads) * a.ring + slot) * a.dim + d;
        float      u = to_f32(src[0]), v = d + 1 < a.dim ? to_f32(src[1]) : 0.f;
        if (d < a.rot_dims) {
            const float c = cs[i], z = sn[i], u2 = u * c - v * z, v2 = v * c + u * z;
            u = u2, v = v2;
        }
        dst[0] = from_f32<E>(u);
        if (d + 1 < a.dim) dst[1] = from_f32<E>(v);
    }
    for (int w = threadIdx.x; w < a.kv_heads * a.vdim; w += blockDim.x) {
        const int g = w / a.vdim, d = w - g * a.vdim;
        slab_rows<E>(s.slab, a.v_off)[((size_t)g * a.ring + slot) * a.vdim + d] = row[a.v_col + w];
    }
}

// The same for bf16 heads of a multiple of 8 dimensions: 16 bytes per access
__global__ void __launch_bounds__(256) window_write8_kernel(const WindowKernelParams p)
{
    using E = __nv_bfloat16;
    __shared__ float cs[kMaxHeadDim / 2], sn[kMaxHeadDim / 2];
    pdl_wait();
    pdl_launch_dependents();
    const WindowAttention& a = p.a;
    const SeqSpan          s = p.c.spans[blockIdx.y];
    if ((int)blockIdx.x >= s.n || !s.live) return;
    const int pos = s.history + blockIdx.x;
    E*        row = static_cast<E*>(p.c.proj) + (size_t)(s.tok0 + blockIdx.x) * p.c.proj_ld;
    for (int i = threadIdx.x; i < a.rot_dims / 2; i += blockDim.x) sincosf((float)pos * a.inv_freq[i], &sn[i], &cs[i]);
    __syncthreads();
    const int slot = pos % a.ring, per = a.dim / 8, per_v = a.vdim / 8;
    const int n_qk = (a.heads + a.kv_heads) * per, total = n_qk + a.kv_heads * per_v;
    for (int w = threadIdx.x; w < total; w += blockDim.x) {
        if (w >= n_qk) {
            const int x = w - n_qk, g = x / per_v, d = (x - g * per_v) * 8;
            *reinterpret_cast<uint4*>(slab_rows<E>(s.slab, a.v_off) + ((size_t)g * a.ring + slot) * a.vdim + d) =
                *reinterpret_cast<const uint4*>(row + a.v_col + g * a.vdim + d);
            continue;
        }
        const int  hh = w / per, d = (w - hh * per) * 8;
        const bool is_q = hh < a.heads;
        if (is_q && d >= a.rot_dims) continue;  // stays where it is
        E*    src = row + (is_q ? a.q_col + hh * a.dim : a.k_col + (hh - a.heads) * a.dim) + d;
        E*    dst = is_q ? src : slab_rows<E>(s.slab, a.k_off) + ((size_t)(hh - a.heads) * a.ring + slot) * a.dim + d;
        uint4 v   = *reinterpret_cast<const uint4*>(src);
        auto  turn = [&](uint32_t x, int i) {
            if (2 * i >= a.rot_dims) return x;
            const float u = bf16_lo(x), y = bf16_hi(x), c = cs[i], z = sn[i];
            return pack_bf16(u * c - y * z, y * c + u * z);
        };
        v.x = turn(v.x, d / 2), v.y = turn(v.y, d / 2 + 1), v.z = turn(v.z, d / 2 + 2), v.w = turn(v.w, d / 2 + 3);
        *reinterpret_cast<uint4*>(dst) = v;
    }
}

// One CTA per (block that this launch completes, kv head, sequence): the mean of its keys and of its values as cached.
template<typename E>
__global__ void __launch_bounds__(128) window_pool_kernel(const WindowKernelParams p)
{
    pdl_wait();
    pdl_launch_dependents();
    const WindowAttention& a = p.a;
    const SeqSpan          s = p.c.spans[blockIdx.z];
    const int              g = blockIdx.y, b = s.history / a.pool + blockIdx.x;
    if (!s.live || (b + 1) * a.pool > s.history + s.n || b >= a.pool_rows) return;
    const float inv = 1.f / (float)a.pool;
    for (int d = threadIdx.x; d < a.dim + a.vdim; d += blockDim.x) {
        const bool is_k = d < a.dim;
        const int  e = is_k ? d : d - a.dim, width = is_k ? a.dim : a.vdim;
        const E*   src = slab_rows<E>(s.slab, is_k ? a.k_off : a.v_off) + (size_t)g * a.ring * width + e;
        float      sum = 0.f;
        for (int j = 0; j < a.pool; ++j) sum += to_f32(src[(size_t)((b * a.pool + j) % a.ring) * width]);
        slab_rows<E>(s.slab, is_k ? a.pk_off : a.pv_off)[((size_t)g * a.pool_rows + b) * width + e] = from_f32<E>(sum * inv);
    }
}

template<typename E>
__device__ __forceinline__ float dot_row(const E* k, const float* q, int dim, bool vec);
template<>
__device__ __forceinline__ float dot_row<float>(const float* k, const float* q, int dim, bool vec)
{
    float s = 0.f;
    if (vec) {
        for (int d = 0; d < dim; d += 4) {
            const float4 x = *reinterpret_cast<const float4*>(k + d);
            s = fmaf(x.x, q[d], s), s = fmaf(x.y, q[d + 1], s), s = fmaf(x.z, q[d + 2], s), s = fmaf(x.w, q[d + 3], s);
        }
    }
    else {
        for (int d = 0; d < dim; ++d) s = fmaf(k[d], q[d], s);
    }
    return s;
}
template<>
__device__ __forceinline__ float dot_row<__nv_bfloat16>(const __nv_bfloat16* k, const float* q, int dim, bool vec)
{
    float s = 0.f;
    if (vec) {
        for (int d = 0; d < dim; d += 8) {
            const uint4 x = *reinterpret_cast<const uint4*>(k + d);
            s = fmaf(bf16_lo(x.x), q[d], s), s = fmaf(bf16_hi(x.x), q[d + 1], s);
            s = fmaf(bf16_lo(x.y), q[d + 2], s), s = fmaf(bf16_hi(x.y), q[d + 3], s);
            s = fmaf(bf16_lo(x.z), q[d + 4], s), s = fmaf(bf16_hi(x.z), q[d + 5], s);
            s = fmaf(bf16_lo(x.w), q[d + 6], s), s = fmaf(bf16_hi(x.w), q[d + 7], s);
        }
    }
    else {
        for (int d = 0; d < dim; ++d) s = fmaf(to_f32(k[d]), q[d], s);
    }
    return s;
}

// One CTA per (query, head, sequence); its warps take tiles of 32 visible keys in turn (lane = key for the scores, lane =
// value dimension for the output), each with an online softmax of its own, merged at the end.
template<typename E, int W>
__global__ void __launch_bounds__(W * 32) window_attention_kernel(const WindowKernelParams p)
{
    __shared__ float q[kMaxHeadDim];
    __shared__ float s_m[W], s_l[W], s_o[W][kMaxHeadDim];
    pdl_wait();
    pdl_launch_dependents();
    const WindowAttention& a = p.a;
    const SeqSpan          s = p.c.spans[blockIdx.z];
    const int              h = blockIdx.y;
    if ((int)blockIdx.x >= s.n || !s.live) return;
    const int    i = s.history + blockIdx.x, t = s.tok0 + blockIdx.x;
    const int    warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const E*     row = static_cast<const E*>(p.c.proj) + (size_t)t * p.c.proj_ld;
    for (int d = threadIdx.x; d < a.dim; d += W * 32) q[d] = to_f32(row[a.q_col + h * a.dim + d]) * a.scale;
    __syncthreads();
    const Visible v     = visible_of(i, a.window, a.pool);
    const int     total = v.blocks + i - v.first + 1;
    const int     g     = h / (a.heads / a.kv_heads);
    const E*      k_tok = slab_rows<E>(s.slab, a.k_off) + (size_t)g * a.ring * a.dim;
    const E*      v_tok = slab_rows<E>(s.slab, a.v_off) + (size_t)g * a.ring * a.vdim;
    const E*      k_blk = slab_rows<E>(s.slab, a.pk_off) + (size_t)g * a.pool_rows * a.dim;
    const E*      v_blk = slab_rows<E>(s.slab, a.pv_off) + (size_t)g * a.pool_rows * a.vdim;
    const bool    vec   = a.dim % (16 / (int)sizeof(E)) == 0;
    float         m = -INFINITY, l = 0.f, o[kMaxHeadDim / 32];
#pragma unroll
    for (int e = 0; e < kMaxHeadDim / 32; ++e) o[e] = 0.f;
    for (int tile = warp * 32; tile < total; tile += W * 32) {
        const int  idx  = tile + lane;
        const bool blk  = idx < v.blocks;
        const int  slot = blk ? idx : (v.first + idx - v.blocks) % a.ring;
        float      sc   = -INFINITY;
        if (idx < total) {
            sc = dot_row<E>((blk ? k_blk : k_tok) + (size_t)slot * a.dim, q, a.dim, vec);
            if (a.softcap > 0.f) sc = a.softcap * tanhf(sc / a.softcap);
        }
        float mx = sc;
#pragma unroll
        for (int x = 16; x >= 1; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
        const float m2 = fmaxf(m, mx), alpha = expf(m - m2), w = expf(sc - m2);
        l = l * alpha + warp_sum(w);
        m = m2;
#pragma unroll
        for (int e = 0; e < kMaxHeadDim / 32; ++e) o[e] *= alpha;
        const int n = min(32, total - tile);
        for (int j = 0; j < n; ++j) {
            const float wj  = __shfl_sync(0xffffffffu, w, j);
            const int   sj  = __shfl_sync(0xffffffffu, slot, j);
            const E*    src = (tile + j < v.blocks ? v_blk : v_tok) + (size_t)sj * a.vdim;
#pragma unroll
            for (int e = 0; e < kMaxHeadDim / 32; ++e) {
                if (lane + 32 * e < a.vdim) o[e] = fmaf(wj, to_f32(src[lane + 32 * e]), o[e]);
            }
        }
    }
    if (lane == 0) s_m[warp] = m, s_l[warp] = l;
#pragma unroll
    for (int e = 0; e < kMaxHeadDim / 32; ++e) s_o[warp][lane + 32 * e] = o[e];
    __syncthreads();
    float top = -INFINITY, sum = 0.f;
    for (int w = 0; w < W; ++w) top = fmaxf(top, s_m[w]);
    for (int w = 0; w < W; ++w) sum += s_l[w] * expf(s_m[w] - top);
    const float gate = sigmoid_f32(to_f32(row[a.g_col + h])) / sum;
    E*          out  = static_cast<E*>(p.c.out) + (size_t)t * p.c.out_ld;
    for (int d = threadIdx.x; d < a.vdim; d += W * 32) {
        float y = 0.f;
        for (int w = 0; w < W; ++w) y += s_o[w][d] * expf(s_m[w] - top);
        out[h * a.vdim + d] = from_f32<E>(y * gate);
    }
    if (h == a.heads - 1) {
        for (int d = a.heads * a.vdim + threadIdx.x; d < p.c.out_pad; d += W * 32) out[d] = from_f32<E>(0.f);
    }
}

bool valid(const WindowAttention& a, const MixerCall& c)
{
    return a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.dim <= kMaxHeadDim && a.vdim > 0
           && a.vdim <= kMaxHeadDim && a.rot_dims >= 0 && a.rot_dims <= a.dim && a.rot_dims % 2 == 0 && a.ring > 0 && a.window >= 0
           && a.pool >= 0 && (a.pool == 0 || (a.window > 0 && a.pool_rows > 0)) && c.batch > 0 && c.max_n > 0 && c.batch <= 65535;
}

template<typename E>
int write_and_pool(tm_handle* h, const WindowKernelParams& p, cudaStream_t st)
{
    const bool wide = sizeof(E) == 2 && p.a.dim % 8 == 0 && p.a.vdim % 8 == 0 && p.c.proj_ld % 8 == 0 && p.a.q_col % 8 == 0 && p.a.k_col % 8 == 0
                      && p.a.v_col % 8 == 0;
    const cudaError_t e = wide ? launch_kernel(window_write8_kernel, dim3(p.c.max_n, p.c.batch), dim3(256), 0, st, p.c.pdl, p) :
                                 launch_kernel(window_write_kernel<E>, dim3(p.c.max_n, p.c.batch), dim3(128), 0, st, p.c.pdl, p);
    if (e != cudaSuccess) return TM_ERR_CUDA;
    ++h->launches;
    if (p.a.pool > 0) {
        const dim3 grid((p.c.max_n + p.a.pool - 1) / p.a.pool, p.a.kv_heads, p.c.batch);
        if (launch_kernel(window_pool_kernel<E>, grid, dim3(128), 0, st, p.c.pdl, p) != cudaSuccess) return TM_ERR_CUDA;
        ++h->launches;
    }
    return TM_OK;
}

template<typename E>
int attend(tm_handle* h, const WindowKernelParams& p, cudaStream_t st)
{
    const dim3 grid(p.c.max_n, p.a.heads, p.c.batch);
    const bool few = (long long)p.c.tokens * p.a.heads < 4 * h->sm_count;
    const cudaError_t e = few ? launch_kernel(window_attention_kernel<E, 16>, grid, dim3(512), 0, st, p.c.pdl, p) :
                                launch_kernel(window_attention_kernel<E, 4>, grid, dim3(128), 0, st, p.c.pdl, p);
    if (e != cudaSuccess) return TM_ERR_CUDA;
    ++h->launches;
    return TM_OK;
}

}  // namespace

int window_attention_write(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st)
{
    if (!valid(a, c)) return TM_ERR_UNSUPPORTED;
    const WindowKernelParams p{a, c};
    return c.f32 ? write_and_pool<float>(h, p, st) : write_and_pool<__nv_bfloat16>(h, p, st);
}

int window_attention_prefill(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st)
{
    const int rc = window_attention_write(h, a, c, st);
    if (rc != TM_OK) return rc;
    const WindowKernelParams p{a, c};
    if (window_attention_tc_supported(a, c)) return window_attention_tc(h, a, c, st);
    return c.f32 ? attend<float>(h, p, st) : attend<__nv_bfloat16>(h, p, st);
}

int window_attention_decode(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st)
{
    if (!valid(a, c)) return TM_ERR_UNSUPPORTED;
    if (window_attention_step_supported(a, c)) return window_attention_step(h, a, c, st);
    const int rc = window_attention_write(h, a, c, st);
    if (rc != TM_OK) return rc;
    const WindowKernelParams p{a, c};
    return c.f32 ? attend<float>(h, p, st) : attend<__nv_bfloat16>(h, p, st);
}

}  // namespace tmb
