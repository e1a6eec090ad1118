// Gated linear attention (GatedLinear in mixers.h).  Per head, with key-channel decay a:
//     S <- diag(a) S + k v^T          o = S^T q
// all of it in fp32.  The columns of S (value channels) never meet: the prefill kernel splits them over lane groups, warps
// and CTAs, while the keys' side (q, a, k) is shared by all columns of a head.  A column is contiguous in memory.
#include "common.cuh"
#include "f32x2.cuh"
#include "gemm_dense.h"
#include "mixers.h"
#include "numeric.cuh"
#include "tm_b200.h"

#include <algorithm>

namespace tmb {
namespace {

constexpr int kMaxDim = 256;

struct LinearParams {
    GatedLinear  d;
    MixerCall    c;
    const float* decay_pre;  // [tokens][heads * dim]
    float*       records;    // [head][token][record]
    float*       o;          // [tokens][heads * vdim]
    int          record;     // floats
    int          chunk;      // tokens of a stage, even
    unsigned*    status;
    long long    max_wait;
};

// sigmoid(z)^(1/tau), by its logarithm
__device__ __forceinline__ float decay_of(float z, float inv_tau)
{
    return expf(-(log1pf(expf(-fabsf(z))) + fmaxf(-z, 0.f)) * inv_tau);
}

int padded_dim(int dim)
{
    int dp = 16;
    while (dp < dim) dp *= 2;
    return dp;
}
int record_floats(const GatedLinear& d)
{
    return 3 * padded_dim(d.dim) + (d.vdim + 3) / 4 * 4;
}

// What the scan reads of a (head, token): scale q | decay | k (DP floats each, zeros beyond dim) | v
template<typename E, int DP>
__global__ void __launch_bounds__(128) linear_gates_kernel(const LinearParams p)
{
    pdl_wait();
    pdl_launch_dependents();
    const GatedLinear& d = p.d;
    const SeqSpan      s = p.c.spans[blockIdx.z];
    const int          h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31, dim = d.dim;
    if (!s.live || (int)blockIdx.x >= s.n || h >= d.heads) return;
    const size_t tok = (size_t)s.tok0 + blockIdx.x;
    const E*     row = static_cast<const E*>(p.c.proj) + tok * p.c.proj_ld;
    const float* pre = p.decay_pre + tok * d.heads * dim + h * dim;
    float*       rec = p.records + ((size_t)h * p.c.tokens + tok) * p.record;
    const float  inv_tau = 1.f / d.tau;
#pragma unroll
    for (int c = lane; c < DP; c += 32) {
        const bool on   = c < dim;
        rec[c]          = on ? to_f32(row[d.q_col + h * dim + c]) * d.scale : 0.f;
        rec[DP + c]     = on ? decay_of(pre[c] + d.bias[h * dim + c], inv_tau) : 0.f;
        rec[2 * DP + c] = on ? to_f32(row[d.k_col + h * dim + c]) : 0.f;
    }
    for (int c = lane; c < p.record - 3 * DP; c += 32) rec[3 * DP + c] = c < d.vdim ? to_f32(row[d.v_col + h * d.vdim + c]) : 0.f;
}

// The same where head sizes are multiples of four: a CTA per token, a thread takes four channels at a time
template<typename E>
__device__ __forceinline__ float4 load4(const E* p)
{
    if constexpr (sizeof(E) == 2) {
        const uint2 w = *reinterpret_cast<const uint2*>(p);
        return make_float4(bf16_lo(w.x), bf16_hi(w.x), bf16_lo(w.y), bf16_hi(w.y));
    }
    else {
        return *reinterpret_cast<const float4*>(p);
    }
}
template<typename E, int DP>
__global__ void __launch_bounds__(256) linear_gates4_kernel(const LinearParams p)
{
    pdl_wait();
    pdl_launch_dependents();
    const GatedLinear& d = p.d;
    const SeqSpan      s = p.c.spans[blockIdx.y];
    if (!s.live || (int)blockIdx.x >= s.n) return;
    const size_t tok = (size_t)s.tok0 + blockIdx.x;
    const E*     row = static_cast<const E*>(p.c.proj) + tok * p.c.proj_ld;
    const float* pre = p.decay_pre + tok * d.heads * d.dim;
    const int    per = p.record / 4;
    const float  inv_tau = 1.f / d.tau;
    for (int x = threadIdx.x; x < d.heads * per; x += 256) {
        const int h = x / per, i = 4 * (x - h * per), part = i < 3 * DP ? i / DP : 3, c = i - part * DP, at = h * d.dim + c;
        float4    y = make_float4(0.f, 0.f, 0.f, 0.f);
        if (part == 3) {
            y = load4(row + d.v_col + h * d.vdim + c);
        }
        else if (c < d.dim) {
            if (part == 1) {
                const float4 z = *reinterpret_cast<const float4*>(pre + at), b = *reinterpret_cast<const float4*>(d.bias + at);
                y = make_float4(decay_of(z.x + b.x, inv_tau), decay_of(z.y + b.y, inv_tau), decay_of(z.z + b.z, inv_tau), decay_of(z.w + b.w, inv_tau));
            }
            else {
                y = load4(row + (part == 0 ? d.q_col : d.k_col) + at);
                if (part == 0) y.x *= d.scale, y.y *= d.scale, y.z *= d.scale, y.w *= d.scale;
            }
        }
        *reinterpret_cast<float4*>(p.records + ((size_t)h * p.c.tokens + tok) * p.record + i) = y;
    }
}

// The sequential part.  CTA = (block of value columns, head, sequence).  Lanes of a group share NC columns; lane `part`
// holds rows [4 part, 4 part + 4) and [DP/2 + 4 part, ...) of each, in pairs.  Records of a head are contiguous, so one bulk
// copy brings a chunk of tokens into a stage.  Tokens go in pairs: their sums are exchanged together, while the next pair is
// under way and the operands of the one behind it are on their way from shared memory.
// NC: columns of a lane group; four use the shared memory best, two spread a short batch over more SMs.
template<int DP, int NC>
struct LinearShape {
    static constexpr int kThreads = 128, kLanes = DP / 8;
    static constexpr int kColumns = kThreads / kLanes * NC;
    static constexpr int kStages  = 3;
    static constexpr int kBits    = kLanes == 2 ? 1 : (kLanes == 4 || NC == 2 ? 2 : 3);  // exchanges that halve the number of sums
};

// A store that the compiler need not order against loads from shared memory, as it has to with an ordinary pointer
// (and no branch around it)
__device__ __forceinline__ void store_global_if(bool on, float* p, float v)
{
    asm volatile(
        "{\n"
        ".reg .pred p;\n"
        "setp.ne.b32 p, %2, 0;\n"
        "@p st.global.f32 [%0], %1;\n"
        "}\n" ::"l"(__cvta_generic_to_global(p)),
        "f"(v), "r"((int)on));
}

template<int DP, int NC>
__global__ void __launch_bounds__(128) linear_scan_kernel(const LinearParams p)
{
    using S = LinearShape<DP, NC>;
    extern __shared__ __align__(128) float sm[];
    __shared__ uint64_t full[S::kStages];
    const int tid = threadIdx.x;
    if (tid == 0) {
        for (int i = 0; i < S::kStages; ++i) mbar_init(&full[i], 1);
        fence_mbar_init();
    }
    __syncthreads();
    pdl_wait();
    pdl_launch_dependents();
    const GatedLinear& d = p.d;
    const SeqSpan      s = p.c.spans[blockIdx.z];
    if (!s.live || s.n <= 0) return;
    const int    h = blockIdx.y, dim = d.dim, vdim = d.vdim, c0 = blockIdx.x * S::kColumns, CH = p.chunk;
    const float* src    = p.records + ((size_t)h * p.c.tokens + s.tok0) * p.record;
    const int    chunks = (s.n + CH - 1) / CH;
    auto fetch = [&](int ch) {
        const int      stage = ch % S::kStages;
        const uint32_t bytes = (uint32_t)min(CH, s.n - ch * CH) * p.record * 4;
        mbar_arrive_expect_tx(&full[stage], bytes);
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                         smem_u32(sm + (size_t)stage * CH * p.record)),
                     "l"(src + (size_t)ch * CH * p.record), "r"(bytes), "r"(smem_u32(&full[stage]))
                     : "memory");
    };
    if (tid == 0) {
        for (int ch = 0; ch < min(S::kStages, chunks); ++ch) fetch(ch);
    }
    constexpr int NV = 2 * NC, kKeep = NV >> S::kBits;
    const int     part = tid % S::kLanes, col0 = c0 + tid / S::kLanes * NC;
    float*        state = reinterpret_cast<float*>(s.slab + d.state_off) + (size_t)h * dim * vdim;
    auto          row_of = [&](int i) { return (i >> 1) * (DP / 2) + 4 * part + 2 * (i & 1); };  // first row of pair i
    f32x2         st[NC][4];
#pragma unroll
    for (int c = 0; c < NC; ++c) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int    r  = row_of(i);
            const float* at = state + (size_t)(col0 + c) * dim + r;
            const bool   on = s.history > 0 && col0 + c < vdim;
            st[c][i]        = pair_of(on && r < dim ? at[0] : 0.f, on && r + 1 < dim ? at[1] : 0.f);
        }
    }
    // sums over the lanes of the group: a lane ends up with numbers [first, first + kKeep) of the pair's (token, column)
    int first = 0;
#pragma unroll
    for (int level = 0; level < S::kBits; ++level) first += ((part >> level) & 1) * (NV >> (level + 1));
    auto scatter_sums = [&](float (&x)[NV]) {
#pragma unroll
        for (int level = 0; level < S::kBits; ++level) {
            const int  half = NV >> (level + 1);
            const bool up   = (part >> level) & 1;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float keep = up ? x[i + half] : x[i], send = up ? x[i] : x[i + half];
                x[i] = keep + __shfl_xor_sync(0xffffffffu, send, 1 << level);
            }
        }
#pragma unroll
        for (int m = 1 << S::kBits; m < S::kLanes; m *= 2) {
#pragma unroll
            for (int i = 0; i < kKeep; ++i) x[i] += __shfl_xor_sync(0xffffffffu, x[i], m);
        }
    };
    float* o_out = p.o + (size_t)s.tok0 * d.heads * vdim + h * vdim + col0;
    int    held = -1;  // first token of the pair whose outputs wait in `sums`
    float  sums[NV] = {};
    bool   held_two = false, ok = true;
    auto store_outputs = [&]() {
        scatter_sums(sums);
        const bool mine = held >= 0 && part < (1 << S::kBits);
#pragma unroll
        for (int i = 0; i < kKeep; ++i) {
            const int b = (first + i) / NC, c = (first + i) % NC;
            store_global_if(mine && (b == 0 || held_two) && col0 + c < vdim, o_out + (size_t)(max(held, 0) + b) * d.heads * vdim + c, sums[i]);
        }
    };
    const int v_at = 3 * DP + (col0 < vdim ? col0 : 0);  // groups beyond the last column write nothing
    struct Pair {
        f32x2 q[2][4], a[2][4], k[2][4];
        float v[2][NC];
    };
    int ch = 0;
    for (; ch < chunks; ++ch) {
        ok           = mbar_wait(&full[ch % S::kStages], (ch / S::kStages) & 1, p.max_wait);
        const int nt = min(CH, s.n - ch * CH);
        const float* const stage = sm + (size_t)(ch % S::kStages) * CH * p.record;
        auto load = [&](int t, Pair& x) {
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const float* rec = stage + (size_t)min(t + j, nt - 1) * p.record;
                auto vec = [&](int which, f32x2 (&y)[4]) {
#pragma unroll
                    for (int q = 0; q < 2; ++q) {
                        const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(rec + which * DP + q * (DP / 2) + 4 * part);
                        y[2 * q] = w.x, y[2 * q + 1] = w.y;
                    }
                };
                vec(0, x.q[j]), vec(1, x.a[j]), vec(2, x.k[j]);
                if constexpr (NC == 4) {
                    const float4 w = *reinterpret_cast<const float4*>(rec + v_at);
                    x.v[j][0] = w.x, x.v[j][1] = w.y, x.v[j][2] = w.z, x.v[j][3] = w.w;
                }
                else {
                    const float2 w = *reinterpret_cast<const float2*>(rec + v_at);
                    x.v[j][0] = w.x, x.v[j][1] = w.y;
                }
            }
        };
        auto token = [&](const Pair& x, int j) {
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const f32x2 v = pair_of(x.v[j][c], x.v[j][c]);
                f32x2       y[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) st[c][i] = fma2(x.a[j][i], st[c][i], mul2(x.k[j][i], v));
#pragma unroll
                for (int i = 0; i < 4; i += 2) y[i] = fma2(x.q[j][i + 1], st[c][i + 1], mul2(x.q[j][i], st[c][i]));
                const float2 f = halves(y[0]), g = halves(y[2]);
                sums[j * NC + c] = (f.x + f.y) + (g.x + g.y);
            }
        };
        Pair now;
        load(0, now);
        int t = 0;
#pragma unroll 2
        for (; t + 1 < nt; t += 2) {
            Pair next;
            load(min(t + 2, nt - 1), next);
            store_outputs();
            token(now, 0);
            token(now, 1);
            held = ch * CH + t, held_two = true;
            now  = next;
        }
        if (t < nt) {  // an odd last token
            store_outputs();
            token(now, 0);
            held = ch * CH + t, held_two = false;
        }
        // everybody is through with the stage; one outcome for the whole CTA
        if (!__syncthreads_and(ok)) break;
        if (tid == 0 && ch + S::kStages < chunks) fetch(ch + S::kStages);
    }
    if (ch < chunks) {
        if (tid == 0) {
            atomicOr(p.status, kStatusGemmPipeWait);
            // not before the copies in flight have landed
            for (int c = ch; c < min(ch + S::kStages, chunks); ++c) mbar_wait(&full[c % S::kStages], (c / S::kStages) & 1, p.max_wait);
        }
        return;
    }
    store_outputs();
#pragma unroll
    for (int c = 0; c < NC; ++c) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int    r   = row_of(i);
            float*       dst = state + (size_t)(col0 + c) * dim + r;
            const float2 f   = halves(st[c][i]);
            if (col0 + c < vdim && r < dim) dst[0] = f.x;
            if (col0 + c < vdim && r + 1 < dim) dst[1] = f.y;
        }
    }
}

__device__ __forceinline__ float silu_f32(float g)
{
    return g * sigmoid_f32(g);
}

// Head outputs over their root mean square, times the norm weight and silu of the gate: a warp per (token, head)
template<typename E>
__global__ void __launch_bounds__(256) linear_finish_kernel(const LinearParams p)
{
    pdl_wait();
    pdl_launch_dependents();
    const GatedLinear& d    = p.d;
    const int          lane = threadIdx.x & 31, t = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5);
    E*                 out  = static_cast<E*>(p.c.out) + (size_t)t * p.c.out_ld;
    if (blockIdx.y == 0) {
        for (int n = d.heads * d.vdim + threadIdx.x; n < p.c.out_pad; n += 256) out[n] = from_f32<E>(0.f);
    }
    if (h >= d.heads) return;
    const float* o   = p.o + ((size_t)t * d.heads + h) * d.vdim;
    const E*     row = static_cast<const E*>(p.c.proj) + (size_t)t * p.c.proj_ld + d.g_col + h * d.vdim;
    float        x[kMaxDim / 32], g[kMaxDim / 32], sq = 0.f;
#pragma unroll
    for (int e = 0; e < kMaxDim / 32; ++e) {
        const int  c  = lane + 32 * e;
        const bool on = c < d.vdim;
        x[e] = on ? o[c] : 0.f, g[e] = on ? to_f32(row[c]) : 0.f;
        sq += x[e] * x[e];
    }
    const float inv = 1.f / sqrtf(warp_sum(sq) / (float)d.vdim + d.norm_eps);
#pragma unroll
    for (int e = 0; e < kMaxDim / 32; ++e) {
        const int c = lane + 32 * e;
        if (c < d.vdim) out[h * d.vdim + c] = from_f32<E>(x[e] * inv * d.norm[c] * silu_f32(g[e]));
    }
}

// One new token per sequence, one CTA per (head, sequence): decay projection, step, head norm and gate in one kernel.  Lanes
// share a column of S as in the scan; the state passes through registers once, and where all of a thread's columns fit
// (HELD) their reads are under way before anything else is known.
constexpr int kHeld = 8;

template<typename E, int DP, bool HELD>
__global__ void __launch_bounds__(256, 2) linear_step_kernel(const LinearParams p)
{
    constexpr int kLanes = DP / 8, kColumns = 256 / kLanes, kPer = 256 / DP, kVec = 16 / sizeof(E);
    __shared__ __align__(16) float a[DP], k[DP], q[DP];
    __shared__ float y[kMaxDim], red[8];
    const GatedLinear& d    = p.d;
    const int          h    = blockIdx.x, dim = d.dim, vdim = d.vdim, n = h * dim;
    const int          tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const SeqSpan      s    = p.c.spans[blockIdx.y];
    const int          part = tid % kLanes, lc = tid / kLanes, passes = (vdim + kColumns - 1) / kColumns;
    float*             state = reinterpret_cast<float*>(s.slab + d.state_off) + (size_t)h * dim * vdim;
    const bool         quad = dim % 4 == 0, old = s.live && s.history > 0;
    float              st[HELD ? kHeld : 1][8];
    auto load = [&](int pass, float (&x)[8]) {
        const int col = pass * kColumns + lc;
#pragma unroll
        for (int b = 0; b < 2; ++b) {
            const int    r0  = b * (DP / 2) + 4 * part;
            const float* src = state + (size_t)col * dim + r0;
            if (old && col < vdim && quad && r0 < dim) {
                const float4 f = __ldcs(reinterpret_cast<const float4*>(src));
                x[4 * b] = f.x, x[4 * b + 1] = f.y, x[4 * b + 2] = f.z, x[4 * b + 3] = f.w;
            }
            else {
#pragma unroll
                for (int e = 0; e < 4; ++e) x[4 * b + e] = old && col < vdim && r0 + e < dim ? src[e] : 0.f;
            }
        }
    };
    // written by this layer's kernel of an earlier step: nothing of this step touches it before
    if (HELD) {
#pragma unroll
        for (int i = 0; i < kHeld; ++i) {
            if (i < passes) load(i, st[HELD ? i : 0]);
        }
    }
    const int  c  = tid / kPer, sub = tid % kPer;
    const bool on = c < dim;
    uint4      w2[4];
    const E*   w2_row = static_cast<const E*>(d.w2) + (size_t)(n + (on ? c : 0)) * d.w2_ld;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = (sub + i * kPer) * kVec;
        w2[i]       = m < d.rank ? *reinterpret_cast<const uint4*>(w2_row + m) : make_uint4(0, 0, 0, 0);
    }
    const float bias = on ? d.bias[n + c] : 0.f, nw = tid < vdim ? d.norm[tid] : 0.f;
    pdl_wait();
    pdl_launch_dependents();
    if (!s.live) return;
    const E*    row = static_cast<const E*>(p.c.proj) + (size_t)s.tok0 * p.c.proj_ld;
    const float kc = on ? to_f32(row[d.k_col + n + c]) : 0.f, qc = on ? to_f32(row[d.q_col + n + c]) * d.scale : 0.f;
    const float gate = tid < vdim ? to_f32(row[d.g_col + h * vdim + tid]) : 0.f;
    float       x = 0.f;
    for (int i = 0;; ++i) {
        const int m = (sub + i * kPer) * kVec;
        if (m >= d.rank) break;
        const uint4 w = i == 0 ? w2[0] : i == 1 ? w2[1] : i == 2 ? w2[2] : i == 3 ? w2[3] : *reinterpret_cast<const uint4*>(w2_row + m);
        const E*    we = reinterpret_cast<const E*>(&w);
        const E*    xe = row + d.a_col + m;
#pragma unroll
        for (int e = 0; e < kVec; ++e) {
            if (m + e < d.rank) x = fmaf(to_f32(we[e]), to_f32(xe[e]), x);
        }
    }
    // the threads of a channel are neighbours; up to 16 of them
#pragma unroll
    for (int m = 1; m < kPer; m *= 2) x += __shfl_xor_sync(0xffffffffu, x, m);
    if (sub == 0 && c < DP) a[c] = on ? decay_of(x + bias, 1.f / d.tau) : 0.f, k[c] = kc, q[c] = qc;
    __syncthreads();
    auto vec = [&](const float* v, float (&f)[8]) {
        const float4 lo = *reinterpret_cast<const float4*>(v + 4 * part), hi = *reinterpret_cast<const float4*>(v + DP / 2 + 4 * part);
        f[0] = lo.x, f[1] = lo.y, f[2] = lo.z, f[3] = lo.w, f[4] = hi.x, f[5] = hi.y, f[6] = hi.z, f[7] = hi.w;
    };
    float aa[8], kk[8], qq[8];
    vec(a, aa), vec(k, kk), vec(q, qq);
    float sq = 0.f;
    auto pass_of = [&](int pass, float (&now)[8]) {
        const int   col = pass * kColumns + lc;
        const float vj  = col < vdim ? to_f32(row[d.v_col + h * vdim + col]) : 0.f;
        float       o   = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            now[i] = fmaf(aa[i], now[i], kk[i] * vj);
            o      = fmaf(qq[i], now[i], o);
        }
#pragma unroll
        for (int m = kLanes / 2; m >= 1; m >>= 1) o += __shfl_xor_sync(0xffffffffu, o, m);
        if (col < vdim) {
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                const int r0  = b * (DP / 2) + 4 * part;
                float*    dst = state + (size_t)col * dim + r0;
                if (quad && r0 < dim) {
                    *reinterpret_cast<float4*>(dst) = make_float4(now[4 * b], now[4 * b + 1], now[4 * b + 2], now[4 * b + 3]);
                }
                else {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        if (r0 + e < dim) dst[e] = now[4 * b + e];
                    }
                }
            }
            if (part == 0) {
                y[col] = o;
                sq += o * o;
            }
        }
    };
    if (HELD) {
#pragma unroll
        for (int i = 0; i < kHeld; ++i) {
            if (i < passes) pass_of(i, st[HELD ? i : 0]);
        }
    }
    else {
        for (int i = 0; i < passes; ++i) {
            load(i, st[0]);
            pass_of(i, st[0]);
        }
    }
    sq = warp_sum(sq);
    if (lane == 0) red[warp] = sq;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) total += red[i];
    const float inv = 1.f / sqrtf(total / (float)vdim + d.norm_eps);
    E*          out = static_cast<E*>(p.c.out) + (size_t)s.tok0 * p.c.out_ld;
    if (tid < vdim) out[h * vdim + tid] = from_f32<E>(y[tid] * inv * nw * silu_f32(gate));
    if (h == d.heads - 1) {
        for (int i = d.heads * vdim + tid; i < p.c.out_pad; i += 256) out[i] = from_f32<E>(0.f);
    }
}

template<int DP, int NC>
cudaError_t scan_kernel_launch(const LinearParams& p, cudaStream_t st)
{
    using S           = LinearShape<DP, NC>;
    const size_t smem = (size_t)S::kStages * p.chunk * p.record * 4;
    const dim3   grid((p.d.vdim + S::kColumns - 1) / S::kColumns, p.d.heads, p.c.batch);
    return launch_kernel(linear_scan_kernel<DP, NC>, grid, dim3(S::kThreads), smem, st, p.c.pdl, p);
}

template<typename E, int DP>
cudaError_t scan_launch(LinearParams p, int sms, cudaStream_t st)
{
    const GatedLinear& d    = p.d;
    const bool         quad = d.dim % 4 == 0 && d.vdim % 4 == 0 && p.c.proj_ld % 4 == 0 && d.q_col % 4 == 0 && d.k_col % 4 == 0 && d.v_col % 4 == 0;
    cudaError_t        e = quad ? launch_kernel(linear_gates4_kernel<E, DP>, dim3(p.c.max_n, p.c.batch), dim3(256), 0, st, p.c.pdl, p) :
                                  launch_kernel(linear_gates_kernel<E, DP>, dim3(p.c.max_n, (d.heads + 3) / 4, p.c.batch), dim3(128), 0, st, p.c.pdl, p);
    if (e != cudaSuccess) return e;
    p.chunk = std::max(2, std::min(16, 16384 / (p.record * 4) / 2 * 2));
    const long long ctas = (long long)((p.d.vdim + LinearShape<DP, 4>::kColumns - 1) / LinearShape<DP, 4>::kColumns) * p.d.heads * p.c.batch;
    return ctas < sms ? scan_kernel_launch<DP, 2>(p, st) : scan_kernel_launch<DP, 4>(p, st);
}

template<typename E, int DP>
cudaError_t step_launch(const LinearParams& p, cudaStream_t st)
{
    const bool held = (p.d.vdim + 2048 / DP - 1) / (2048 / DP) <= kHeld;
    return launch_kernel(held ? linear_step_kernel<E, DP, true> : linear_step_kernel<E, DP, false>, dim3(p.d.heads, p.c.batch), dim3(256), 0, st, p.c.pdl, p);
}

template<typename E>
cudaError_t dispatch(const LinearParams& p, bool step, int sms, cudaStream_t st)
{
    switch (padded_dim(p.d.dim)) {
        case 16: return step ? step_launch<E, 16>(p, st) : scan_launch<E, 16>(p, sms, st);
        case 32: return step ? step_launch<E, 32>(p, st) : scan_launch<E, 32>(p, sms, st);
        case 64: return step ? step_launch<E, 64>(p, st) : scan_launch<E, 64>(p, sms, st);
        case 128: return step ? step_launch<E, 128>(p, st) : scan_launch<E, 128>(p, sms, st);
        default: return step ? step_launch<E, 256>(p, st) : scan_launch<E, 256>(p, sms, st);
    }
}

bool valid(const GatedLinear& d, const MixerCall& c)
{
    return d.heads > 0 && d.heads <= 65535 && d.dim > 0 && d.dim <= kMaxDim && d.vdim > 0 && d.vdim <= kMaxDim && d.rank > 0 && d.tau > 0.f && c.batch > 0
           && c.batch <= 65535 && c.tokens > 0;
}

cudaError_t prepare(int)
{
    constexpr int smem = 3 * 16384;  // at most: a chunk of several tokens fits 16 KB, and two tokens take no more
    cudaError_t   e    = cudaSuccess;
    for (const void* f : {(const void*)linear_scan_kernel<16, 2>, (const void*)linear_scan_kernel<32, 2>, (const void*)linear_scan_kernel<64, 2>,
                          (const void*)linear_scan_kernel<128, 2>, (const void*)linear_scan_kernel<256, 2>, (const void*)linear_scan_kernel<16, 4>,
                          (const void*)linear_scan_kernel<32, 4>, (const void*)linear_scan_kernel<64, 4>, (const void*)linear_scan_kernel<128, 4>,
                          (const void*)linear_scan_kernel<256, 4>}) {
        if (e == cudaSuccess) e = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    }
    return e;
}
const KernelPreparation g_prepare(prepare);

}  // namespace

// decay pre-activations and outputs, to a multiple of four floats each; behind them the records
size_t gated_linear_scratch_floats(const GatedLinear& d)
{
    return (size_t)(d.heads * d.dim + 3) / 4 * 4 + (size_t)(d.heads * d.vdim + 3) / 4 * 4 + (size_t)d.heads * record_floats(d);
}

int gated_linear_prefill(tm_handle* h, const GatedLinear& d, const MixerCall& c, float* scratch, cudaStream_t st)
{
    if (!valid(d, c) || !scratch) return TM_ERR_UNSUPPORTED;
    DenseGemm g;
    g.w = d.w2, g.ldw = d.w2_ld;
    g.x = static_cast<const char*>(c.proj) + (size_t)d.a_col * (c.f32 ? 4 : 2), g.ldx = c.proj_ld;
    g.tokens = c.tokens, g.n_out = d.heads * d.dim, g.k = d.rank;
    g.ep.kind = DenseKind::kF32, g.ep.out = scratch, g.ep.out_ld = d.heads * d.dim;
    const int rc = dense_gemm(h, g, c.f32, st, c.pdl);
    if (rc != TM_OK) return rc;
    float* const       o       = scratch + (size_t)c.tokens * ((d.heads * d.dim + 3) / 4 * 4);
    float* const       records = o + (size_t)c.tokens * ((d.heads * d.vdim + 3) / 4 * 4);
    const LinearParams p{d, c, scratch, records, o, record_floats(d), 0, h->status, kMaxWaitCycles};
    cudaError_t        e = c.f32 ? dispatch<float>(p, false, h->sm_count, st) : dispatch<__nv_bfloat16>(p, false, h->sm_count, st);
    const dim3         grid(c.tokens, (d.heads + 7) / 8);
    if (e == cudaSuccess) e = launch_kernel(c.f32 ? linear_finish_kernel<float> : linear_finish_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, c.pdl, p);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    h->launches += 3;
    return TM_OK;
}

int gated_linear_decode(tm_handle* h, const GatedLinear& d, const MixerCall& c, cudaStream_t st)
{
    if (!valid(d, c)) return TM_ERR_UNSUPPORTED;
    const LinearParams p{d, c, nullptr, nullptr, nullptr, 0, 0, h->status, kMaxWaitCycles};
    const cudaError_t  e = c.f32 ? dispatch<float>(p, true, h->sm_count, st) : dispatch<__nv_bfloat16>(p, true, h->sm_count, st);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    ++h->launches;
    return TM_OK;
}

}  // namespace tmb
