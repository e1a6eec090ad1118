// Recurrence with a generalised delta rule (DeltaRule in mixers.h).  Per head, with key-channel decay w, removal rate a and
// unit key u = k / |k|:
//     S <- diag(w) S - (a u) (u^T S) + k v^T          o = S^T r
// (both terms read the old S), all of it in fp32.  The columns of S (value channels) never meet, which is what the
// prefill kernel splits over lanes, warps and CTAs; the keys' side (u, a u, w, k, r) is shared by all columns of a head.
#include "common.cuh"
#include "gemm_dense.h"
#include "mixers.h"
#include "numeric.cuh"
#include "tm_b200.h"

namespace tmb {
namespace {

constexpr int kMaxDim    = 256;
constexpr int kChunk     = 16;   // tokens staged in shared memory at a time
constexpr int kPrepWarps = 4;    // warps that stage the next chunk while the others walk through this one

struct DeltaKernelParams {
    DeltaRule    d;
    MixerCall    c;
    const float* decay_pre;
    float*       o;
    int          column_parts;
};

// DP: head size rounded up to 16, 32, ..., 256.  A group of DP / 8 lanes owns a column of S, eight rows per lane in
// registers.
template<int DP>
struct ScanShape {
    static constexpr int kLanes    = DP / 8;
    static constexpr int kThreads  = 256;                 // scanning threads
    static constexpr int kColumns  = kThreads / kLanes;   // columns of one CTA
    static constexpr int kSmem     = 2 * kChunk * (5 * DP + kColumns) * 4;
};

template<typename E, int DP>
__global__ void __launch_bounds__(ScanShape<DP>::kThreads + kPrepWarps * 32) delta_scan_kernel(const DeltaKernelParams p)
{
    using S = ScanShape<DP>;
    extern __shared__ __align__(16) float sm[];  // [2][kChunk][5][DP] u, a u, w, k, r; then [2][kChunk][columns] v
    float* const sm_v = sm + 2 * kChunk * 5 * DP;
    pdl_wait();
    pdl_launch_dependents();
    const DeltaRule& d = p.d;
    const SeqSpan    s = p.c.spans[blockIdx.z];
    if (!s.live || s.n <= 0) return;
    const int  h = blockIdx.y, dim = d.dim, c0 = blockIdx.x * S::kColumns;
    const int  tid = threadIdx.x;
    const bool scan = tid < S::kThreads;
    const E*   proj = static_cast<const E*>(p.c.proj) + (size_t)s.tok0 * p.c.proj_ld;

    // the keys' side of one chunk: a warp per token
    auto stage = [&](int chunk, int buf) {
        const int warp = (tid - S::kThreads) >> 5, lane = tid & 31;
        for (int t = warp; t < kChunk; t += kPrepWarps) {
            const int tok = chunk * kChunk + t;
            if (tok >= s.n) break;
            const E*     row = proj + (size_t)tok * p.c.proj_ld;
            const float* pre = p.decay_pre + (size_t)(s.tok0 + tok) * d.heads * dim + h * dim;
            float*       dst = sm + (size_t)(buf * kChunk + t) * 5 * DP;
            float        k[DP / 32 + 1], ksq = 0.f;
#pragma unroll
            for (int e = 0; e < (DP + 31) / 32; ++e) {
                const int c = lane + 32 * e;
                k[e]        = c < dim ? to_f32(row[d.k_col + h * dim + c]) : 0.f;
                ksq += k[e] * k[e];
            }
            const float inv = 1.f / sqrtf(warp_sum(ksq) + d.unit_eps);
#pragma unroll
            for (int e = 0; e < (DP + 31) / 32; ++e) {
                const int c = lane + 32 * e;
                if (c >= DP) continue;
                float u = 0.f, au = 0.f, w = 0.f, r = 0.f;
                if (c < dim) {
                    u  = k[e] * inv;
                    au = sigmoid_f32(to_f32(row[d.a_col + h * dim + c]) + d.a_bias[h * dim + c]) * u;
                    w  = expf(-d.decay_scale * sigmoid_f32(pre[c] + d.w0[h * dim + c]));
                    r  = to_f32(row[d.r_col + h * dim + c]);
                }
                dst[c] = u, dst[DP + c] = au, dst[2 * DP + c] = w, dst[3 * DP + c] = k[e], dst[4 * DP + c] = r;
            }
            float* vd = sm_v + (size_t)(buf * kChunk + t) * S::kColumns;
            for (int j = lane; j < S::kColumns; j += 32) vd[j] = c0 + j < dim ? to_f32(row[d.v_col + h * dim + c0 + j]) : 0.f;
        }
    };

    // lane's rows of its column: 4 at 4 * part and 4 at DP / 2 + 4 * part (conflict-free 16-byte reads)
    const int part = tid % S::kLanes, lc = tid / S::kLanes, col = c0 + lc;
    float*    state = reinterpret_cast<float*>(s.slab + d.state_off) + (size_t)h * dim * dim;
    float     st[8];
    auto      row_of = [&](int i) { return (i < 4 ? 0 : DP / 2) + 4 * part + (i & 3); };
    if (scan) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int r = row_of(i);
            st[i]       = s.history > 0 && r < dim && col < dim ? state[(size_t)r * dim + col] : 0.f;
        }
    }
    else {
        stage(0, 0);
    }
    __syncthreads();
    const int chunks = (s.n + kChunk - 1) / kChunk;
    for (int ch = 0; ch < chunks; ++ch) {
        const int buf = ch & 1;
        if (scan) {
            const int nt = min(kChunk, s.n - ch * kChunk);
            for (int t = 0; t < nt; ++t) {
                const float* src = sm + (size_t)(buf * kChunk + t) * 5 * DP + 4 * part;
                auto vec = [&](int which, float (&x)[8]) {
                    const float4 lo = *reinterpret_cast<const float4*>(src + which * DP);
                    const float4 hi = *reinterpret_cast<const float4*>(src + which * DP + DP / 2);
                    x[0] = lo.x, x[1] = lo.y, x[2] = lo.z, x[3] = lo.w, x[4] = hi.x, x[5] = hi.y, x[6] = hi.z, x[7] = hi.w;
                };
                float u[8], au[8], w[8], k[8], r[8];
                vec(0, u), vec(1, au), vec(2, w), vec(3, k), vec(4, r);
                const float v = sm_v[(size_t)(buf * kChunk + t) * S::kColumns + lc];
                float       z = 0.f;
#pragma unroll
                for (int i = 0; i < 8; ++i) z = fmaf(u[i], st[i], z);
#pragma unroll
                for (int m = S::kLanes / 2; m >= 1; m >>= 1) z += __shfl_xor_sync(0xffffffffu, z, m);
                float o = 0.f;
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    st[i] = fmaf(w[i], st[i], fmaf(k[i], v, -au[i] * z));
                    o     = fmaf(r[i], st[i], o);
                }
#pragma unroll
                for (int m = S::kLanes / 2; m >= 1; m >>= 1) o += __shfl_xor_sync(0xffffffffu, o, m);
                if (part == 0 && col < dim) p.o[(size_t)(s.tok0 + ch * kChunk + t) * d.heads * dim + h * dim + col] = o;
            }
        }
        else if (ch + 1 < chunks) {
            stage(ch + 1, buf ^ 1);
        }
        __syncthreads();
    }
    if (scan) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int r = row_of(i);
            if (r < dim && col < dim) state[(size_t)r * dim + col] = st[i];
        }
    }
}

// Head outputs over their root mean square, times the norm weight and the output gate: one warp per (token, head)
template<typename E>
__global__ void __launch_bounds__(256) delta_finish_kernel(const DeltaKernelParams p)
{
    pdl_wait();
    pdl_launch_dependents();
    const DeltaRule& d    = p.d;
    const int        lane = threadIdx.x & 31, t = blockIdx.x;
    const E*         row  = static_cast<const E*>(p.c.proj) + (size_t)t * p.c.proj_ld;
    E*               out  = static_cast<E*>(p.c.out) + (size_t)t * p.c.out_ld;
    for (int h = threadIdx.x >> 5; h < d.heads; h += 8) {
        const float* o  = p.o + ((size_t)t * d.heads + h) * d.dim;
        float        sq = 0.f;
        for (int c = lane; c < d.dim; c += 32) sq += o[c] * o[c];
        const float inv = 1.f / sqrtf(warp_sum(sq) / (float)d.dim + d.norm_eps);
        for (int c = lane; c < d.dim; c += 32) {
            const int n = h * d.dim + c;
            out[n]      = from_f32<E>(o[c] * inv * d.norm[n] * sigmoid_f32(to_f32(row[d.g_col + n])));
        }
    }
    for (int n = d.heads * d.dim + threadIdx.x; n < p.c.out_pad; n += 256) out[n] = from_f32<E>(0.f);
}

// One new token per sequence, one CTA per (head, sequence): decay projection, step, head norm and gate in one kernel.
// The state passes through registers once: thread = (column, every RG-th row).
// ROWS: state elements per thread, held in registers between the two products; 0: read again for the second (large heads).
template<typename E, int ROWS, int kStepThreads>
__global__ void __launch_bounds__(kStepThreads) delta_step_kernel(const DeltaKernelParams p)
{
    __shared__ float u[kMaxDim], au[kMaxDim], w[kMaxDim], k[kMaxDim], r[kMaxDim], v[kMaxDim];
    __shared__ float red[kStepThreads], zs[kMaxDim], warp_red[kStepThreads / 32];
    const DeltaRule& d   = p.d;
    const int        h   = blockIdx.x, dim = d.dim;
    const int        tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait();
    pdl_launch_dependents();
    const SeqSpan s = p.c.spans[blockIdx.y];
    if (!s.live) return;
    const int    groups = kStepThreads / dim;  // row groups; dim <= 256 leaves at least two
    const int    col = tid % dim, rg = tid / dim;
    const bool   on  = rg < groups;
    float*       state = reinterpret_cast<float*>(s.slab + d.state_off) + (size_t)h * dim * dim;
    float        st[ROWS > 0 ? ROWS : 1];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int row = rg + i * groups;
        st[i]         = on && row < dim && s.history > 0 ? state[(size_t)row * dim + col] : 0.f;
    }
    const E* row = static_cast<const E*>(p.c.proj) + (size_t)s.tok0 * p.c.proj_ld;
    float    ksq = 0.f;
    for (int c = tid; c < dim; c += kStepThreads) {
        k[c] = to_f32(row[d.k_col + h * dim + c]);
        v[c] = to_f32(row[d.v_col + h * dim + c]);
        r[c] = to_f32(row[d.r_col + h * dim + c]);
        ksq += k[c] * k[c];
    }
    ksq = warp_sum(ksq);
    if (lane == 0) warp_red[warp] = ksq;
    // decay: w2 . tanh(w1 h), a warp per channel
    const E* w1 = row + d.w1_col;
    for (int c = warp; c < dim; c += kStepThreads / 32) {
        const E* w2 = static_cast<const E*>(d.w2) + (size_t)(h * dim + c) * d.w2_ld;
        float    x  = 0.f;
        for (int m = lane; m < d.rank; m += 32) x = fmaf(to_f32(w2[m]), to_f32(w1[m]), x);
        x = warp_sum(x);
        if (lane == 0) w[c] = expf(-d.decay_scale * sigmoid_f32(x + d.w0[h * dim + c]));
    }
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) total += warp_red[i];
    const float inv = 1.f / sqrtf(total + d.unit_eps);
    for (int c = tid; c < dim; c += kStepThreads) {
        u[c]  = k[c] * inv;
        au[c] = sigmoid_f32(to_f32(row[d.a_col + h * dim + c]) + d.a_bias[h * dim + c]) * u[c];
    }
    __syncthreads();
    float z = 0.f;
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int x = rg + i * groups;
        if (x < dim) z = fmaf(u[x], st[i], z);
    }
    if (ROWS == 0 && on && s.history > 0) {
        for (int x = rg; x < dim; x += groups) z = fmaf(u[x], state[(size_t)x * dim + col], z);
    }
    red[tid] = on ? z : 0.f;
    __syncthreads();
    if (tid < dim) {
        float x = 0.f;
        for (int g = 0; g < groups; ++g) x += red[g * dim + tid];
        zs[tid] = x;
    }
    __syncthreads();
    float o = 0.f;
    if (on) {
        z = zs[col];
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const int x = rg + i * groups;
            if (x < dim) {
                st[i] = fmaf(w[x], st[i], fmaf(k[x], v[col], -au[x] * z));
                o     = fmaf(r[x], st[i], o);
                state[(size_t)x * dim + col] = st[i];
            }
        }
        if (ROWS == 0) {
            for (int x = rg; x < dim; x += groups) {
                const float old = s.history > 0 ? state[(size_t)x * dim + col] : 0.f;
                const float now = fmaf(w[x], old, fmaf(k[x], v[col], -au[x] * z));
                o               = fmaf(r[x], now, o);
                state[(size_t)x * dim + col] = now;
            }
        }
    }
    red[tid] = on ? o : 0.f;
    __syncthreads();
    float y = 0.f;
    if (tid < dim) {
        for (int g = 0; g < groups; ++g) y += red[g * dim + tid];
    }
    const float sq = warp_sum(y * y);
    if (lane == 0) warp_red[warp] = sq;
    __syncthreads();
    total = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) total += warp_red[i];
    const float rms = 1.f / sqrtf(total / (float)dim + d.norm_eps);
    E*          out = static_cast<E*>(p.c.out) + (size_t)s.tok0 * p.c.out_ld;
    if (tid < dim) {
        const int n = h * dim + tid;
        out[n]      = from_f32<E>(y * rms * d.norm[n] * sigmoid_f32(to_f32(row[d.g_col + n])));
    }
    if (h == d.heads - 1) {
        for (int n = d.heads * dim + tid; n < p.c.out_pad; n += kStepThreads) out[n] = from_f32<E>(0.f);
    }
}

template<typename E, int DP>
cudaError_t scan_launch(DeltaKernelParams p, cudaStream_t st)
{
    using S = ScanShape<DP>;
    cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<E, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::kSmem);
    if (e != cudaSuccess) return e;
    const dim3 grid((p.d.dim + S::kColumns - 1) / S::kColumns, p.d.heads, p.c.batch);
    return launch_kernel(delta_scan_kernel<E, DP>, grid, dim3(S::kThreads + kPrepWarps * 32), S::kSmem, st, p.c.pdl, p);
}

template<typename E>
cudaError_t scan_dispatch(const DeltaKernelParams& p, cudaStream_t st)
{
    if (p.d.dim <= 16) return scan_launch<E, 16>(p, st);
    if (p.d.dim <= 32) return scan_launch<E, 32>(p, st);
    if (p.d.dim <= 64) return scan_launch<E, 64>(p, st);
    if (p.d.dim <= 128) return scan_launch<E, 128>(p, st);
    return scan_launch<E, 256>(p, st);
}

template<typename E>
cudaError_t step_dispatch(const DeltaKernelParams& p, cudaStream_t st)
{
    const dim3 grid(p.d.heads, p.c.batch);
    auto       rows = [&](int threads) { return (p.d.dim + threads / p.d.dim - 1) / (threads / p.d.dim); };
    if (rows(512) <= 8) return launch_kernel(delta_step_kernel<E, 8, 512>, grid, dim3(512), 0, st, p.c.pdl, p);
    if (rows(1024) <= 19) return launch_kernel(delta_step_kernel<E, 19, 1024>, grid, dim3(1024), 0, st, p.c.pdl, p);
    return launch_kernel(delta_step_kernel<E, 0, 1024>, grid, dim3(1024), 0, st, p.c.pdl, p);
}

bool valid(const DeltaRule& d, const MixerCall& c)
{
    return d.heads > 0 && d.heads <= 65535 && d.dim > 0 && d.dim <= kMaxDim && d.rank > 0 && c.batch > 0 && c.batch <= 65535 && c.tokens > 0;
}

}  // namespace

int delta_rule_prefill(tm_handle* h, const DeltaRule& d, const MixerCall& c, float* decay_pre, float* o, cudaStream_t st)
{
    if (!valid(d, c) || !decay_pre || !o) return TM_ERR_UNSUPPORTED;
    const size_t esz = c.f32 ? 4 : 2;
    DenseGemm    g;
    g.w = d.w2, g.ldw = d.w2_ld;
    g.x = static_cast<const char*>(c.proj) + d.w1_col * esz, g.ldx = c.proj_ld;
    g.tokens = c.tokens, g.n_out = d.heads * d.dim, g.k = d.rank;
    g.ep.kind = DenseKind::kF32, g.ep.out = decay_pre, g.ep.out_ld = d.heads * d.dim;
    const int rc = dense_gemm(h, g, c.f32, st, c.pdl);
    if (rc != TM_OK) return rc;
    const DeltaKernelParams p{d, c, decay_pre, o, 0};
    cudaError_t             e = c.f32 ? scan_dispatch<float>(p, st) : scan_dispatch<__nv_bfloat16>(p, st);
    if (e == cudaSuccess) {
        e = c.f32 ? launch_kernel(delta_finish_kernel<float>, dim3(c.tokens), dim3(256), 0, st, c.pdl, p) :
                    launch_kernel(delta_finish_kernel<__nv_bfloat16>, dim3(c.tokens), dim3(256), 0, st, c.pdl, p);
    }
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    h->launches += 2;
    return TM_OK;
}

int delta_rule_decode(tm_handle* h, const DeltaRule& d, const MixerCall& c, cudaStream_t st)
{
    if (!valid(d, c)) return TM_ERR_UNSUPPORTED;
    const DeltaKernelParams p{d, c, nullptr, nullptr, 0};
    const cudaError_t       e = c.f32 ? step_dispatch<float>(p, st) : step_dispatch<__nv_bfloat16>(p, st);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    ++h->launches;
    return TM_OK;
}

}  // namespace tmb
