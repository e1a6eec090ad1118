// Recurrence with a generalised delta rule (DeltaRule in mixers.h).  Per head, with key-channel decay w, removal rate a and
// unit key u = k / |k|:
//     S <- diag(w) S - (a u) (u^T S) + k v^T          o = S^T r
// (both terms read the old S), all of it in fp32.  The columns of S (value channels) never meet, which is what the
// prefill kernel splits over lanes, warps and CTAs; the keys' side (u, a u, w, k, r) is shared by all columns of a head.
// A column is contiguous in memory.
#include "common.cuh"
#include "f32x2.cuh"
#include "gemm_dense.h"
#include "mixers.h"
#include "numeric.cuh"
#include "tm_b200.h"

namespace tmb {
namespace {

constexpr int kMaxDim = 256;

struct DeltaKernelParams {
    DeltaRule    d;
    MixerCall    c;
    const float* decay_pre;  // [tokens][heads * dim]
    float*       records;    // [head][token][record]
    float*       o;          // [tokens][heads * dim], over decay_pre, which nobody needs by then
    unsigned*    status;
    long long    max_wait;
};

// DP: head size rounded up to 32, 64, 128 or 256 in the prefill, from 16 on in the step.
// What the scan reads of a (head, token), made by delta_gates_kernel (b = a u):
//   u (first token of a pair) or u * w of the token before (second)  |  -b  |  w  |  k  |  r  |  v  |  beta, kappa
// Tokens go in pairs, counted from the start of the span.  With z = u^T S read before the token's own update, the second
// token's z follows from the state before the FIRST one:
//   z1 = (u1 * w0)^T S - (u1 . b0) z0 + (u1 . k0) v0 = ... - beta z0 + kappa v0
// so that both products with the state are in flight together.
template<int DP>
struct ScanShape {
    static constexpr int kRows    = DP == 256 ? 8 : 4;    // rows of S per lane
    static constexpr int kLanes   = DP / kRows;           // lanes that share columns
    static constexpr int kPerLane = DP == 256 ? 2 : 4;    // columns of a lane (all lanes of a group have the same ones)
    static constexpr int kThreads = 128;
    static constexpr int kColumns = kThreads / kLanes * kPerLane;  // columns of one CTA
    static constexpr int kRecord  = 6 * DP + 4;                    // floats
    static constexpr int kChunk   = DP <= 64 ? 16 : (DP == 128 ? 8 : 4);  // tokens of a stage
    static constexpr int kStages  = 3;
    static constexpr int kSmem    = kStages * kChunk * kRecord * 4;
};

// one warp per (pair of tokens, head)
template<typename E, int DP>
__global__ void __launch_bounds__(128) delta_gates_kernel(const DeltaKernelParams p)
{
    using S           = ScanShape<DP>;
    constexpr int kPer = (DP + 31) / 32;
    pdl_wait();
    pdl_launch_dependents();
    const DeltaRule& d = p.d;
    const SeqSpan    s = p.c.spans[blockIdx.z];
    const int        h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31, dim = d.dim;
    const int        t0 = 2 * (int)blockIdx.x;
    if (!s.live || t0 >= s.n || h >= d.heads) return;
    const int n = h * dim;
    float     w0[kPer], b0[kPer], k0[kPer];
#pragma unroll
    for (int t = 0; t < 2; ++t) {
        if (t0 + t >= s.n) return;
        const size_t tok = (size_t)s.tok0 + t0 + t;
        const E*     row = static_cast<const E*>(p.c.proj) + tok * p.c.proj_ld;
        const float* pre = p.decay_pre + tok * d.heads * dim + n;
        float        k[kPer], a[kPer], z[kPer], r[kPer], v[kPer], ksq = 0.f;
#pragma unroll
        for (int e = 0; e < kPer; ++e) {
            const int  c  = lane + 32 * e;
            const bool on = c < dim;
            k[e] = on ? to_f32(row[d.k_col + n + c]) : 0.f;
            a[e] = on ? to_f32(row[d.a_col + n + c]) + d.a_bias[n + c] : 0.f;
            z[e] = on ? pre[c] + d.w0[n + c] : 0.f;
            r[e] = on ? to_f32(row[d.r_col + n + c]) : 0.f;
            v[e] = on ? to_f32(row[d.v_col + n + c]) : 0.f;
            ksq += k[e] * k[e];
        }
        const float inv   = 1.f / sqrtf(warp_sum(ksq) + d.unit_eps);
        float       beta = 0.f, kappa = 0.f;
        float*      rec = p.records + ((size_t)h * p.c.tokens + tok) * S::kRecord;
#pragma unroll
        for (int e = 0; e < kPer; ++e) {
            const int   c = lane + 32 * e;
            const float u = k[e] * inv, b = sigmoid_f32(a[e]) * u, w = expf(-d.decay_scale * sigmoid_f32(z[e]));
            float       first = u;
            if (t == 1) {
                beta += u * b0[e];
                kappa += u * k0[e];
                first = u * w0[e];
            }
            if (c < DP) rec[c] = first, rec[DP + c] = -b, rec[2 * DP + c] = w, rec[3 * DP + c] = k[e], rec[4 * DP + c] = r[e], rec[5 * DP + c] = v[e];
            w0[e] = w, b0[e] = b, k0[e] = k[e];
        }
        if (t == 1) {
            beta  = warp_sum(beta);
            kappa = warp_sum(kappa);
        }
        if (lane == 0) *reinterpret_cast<float4*>(rec + 6 * DP) = make_float4(beta, kappa, 0.f, 0.f);
    }
}

// The sequential part.  CTA = (block of value columns, head, sequence); the records of a head are contiguous, so one bulk
// copy brings a chunk of tokens into a stage.
template<int DP>
__global__ void __launch_bounds__(ScanShape<DP>::kThreads) delta_scan_kernel(const DeltaKernelParams p)
{
    using S = ScanShape<DP>;
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
    const DeltaRule& d = p.d;
    const SeqSpan    s = p.c.spans[blockIdx.z];
    if (!s.live || s.n <= 0) return;
    const int    h = blockIdx.y, dim = d.dim, c0 = blockIdx.x * S::kColumns;
    const float* src    = p.records + ((size_t)h * p.c.tokens + s.tok0) * S::kRecord;
    const int    chunks = (s.n + S::kChunk - 1) / S::kChunk;
    auto fetch = [&](int ch) {
        const int      stage = ch % S::kStages;
        const uint32_t bytes = (uint32_t)min(S::kChunk, s.n - ch * S::kChunk) * S::kRecord * 4;
        mbar_arrive_expect_tx(&full[stage], bytes);
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                         smem_u32(sm + (size_t)stage * S::kChunk * S::kRecord)),
                     "l"(src + (size_t)ch * S::kChunk * S::kRecord), "r"(bytes), "r"(smem_u32(&full[stage]))
                     : "memory");
    };
    if (tid == 0) {
        for (int ch = 0; ch < min(S::kStages, chunks); ++ch) fetch(ch);
    }
    // Lanes of a group (kLanes of them) share kPerLane columns; lane `part` holds rows [part * kRows, ...) of each, in pairs.
    constexpr int R2 = S::kRows / 2, NC = S::kPerLane, NV = 2 * NC, kBits = NV == 8 ? 3 : 2;
    const int     part = tid % S::kLanes, col0 = c0 + tid / S::kLanes * NC, row0 = part * S::kRows;
    float*        state = reinterpret_cast<float*>(s.slab + d.state_off) + (size_t)h * dim * dim;
    f32x2         st[NC][R2];
#pragma unroll
    for (int c = 0; c < NC; ++c) {
#pragma unroll
        for (int i = 0; i < R2; ++i) {
            const int    r   = row0 + 2 * i;
            const float* at  = state + (size_t)(col0 + c) * dim + r;
            const bool   on  = s.history > 0 && col0 + c < dim;
            st[c][i]         = pair_of(on && r < dim ? at[0] : 0.f, on && r + 1 < dim ? at[1] : 0.f);
        }
    }
    // A lane ends up with one of the NV = 2 x NC sums of a pair of tokens: token `b0`, column `mine`
    const int b0 = part & 1, mine = NC == 4 ? ((part >> 1) & 1) * 2 + ((part >> 2) & 1) : (part >> 1) & 1;
    // sums over the lanes of the group of x[0..NV): each lane gets sum number b0 * NC + mine
    auto scatter_sums = [&](float (&x)[NV]) {
#pragma unroll
        for (int level = 0; level < kBits; ++level) {
            const int  half = NV >> (level + 1);
            const bool up   = (part >> level) & 1;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float keep = up ? x[i + half] : x[i], send = up ? x[i] : x[i + half];
                x[i] = keep + __shfl_xor_sync(0xffffffffu, send, 1 << level);
            }
        }
#pragma unroll
        for (int m = 1 << kBits; m < S::kLanes; m *= 2) x[0] += __shfl_xor_sync(0xffffffffu, x[0], m);
        return x[0];
    };
    float* o_out = p.o + (size_t)s.tok0 * d.heads * dim + h * dim + col0 + mine;
    int    v_at[NC], held = -1;  // held: first token of the pair whose outputs wait in `sums`
    float  sums[NV] = {};
    bool   held_two = false, ok = true;
#pragma unroll
    for (int c = 0; c < NC; ++c) v_at[c] = 5 * DP + min(col0 + c, DP - 1);
    auto store_outputs = [&]() {
        const float o = scatter_sums(sums);
        if (held >= 0 && part < NV && (b0 == 0 || held_two) && col0 + mine < dim) o_out[(size_t)(held + b0) * d.heads * dim] = o;
    };
    int ch = 0;
    for (; ch < chunks; ++ch) {
        ok           = mbar_wait(&full[ch % S::kStages], (ch / S::kStages) & 1, p.max_wait);
        const int nt = min(S::kChunk, s.n - ch * S::kChunk);
        for (int t = 0; t < nt; t += 2) {
            const bool   two  = t + 1 < nt;
            const float* rec  = sm + (size_t)((ch % S::kStages) * S::kChunk + t) * S::kRecord;
            const float* rec1 = two ? rec + S::kRecord : rec;
            auto vec = [&](const float* r, int which, f32x2 (&x)[R2]) {
#pragma unroll
                for (int i = 0; i < R2; i += 2) {
                    const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(r + which * DP + row0 + 2 * i);
                    x[i] = q.x, x[i + 1] = q.y;
                }
            };
            auto dots = [&](const f32x2 (&x)[R2], float* out) {
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    f32x2 a = mul2(x[0], st[c][0]);
#pragma unroll
                    for (int i = 1; i < R2; ++i) a = fma2(x[i], st[c][i], a);
                    const float2 f = halves(a);
                    out[c]         = f.x + f.y;
                }
            };
            // everything the pair needs from shared memory is on its way before the first sum
            f32x2 x0[R2], x1[R2], b[2][R2], w[2][R2], k[2][R2], r0[R2], r1[R2];
            float v[2][NC], z[NV];
            vec(rec, 0, x0), vec(rec1, 0, x1);
            vec(rec, 1, b[0]), vec(rec, 2, w[0]), vec(rec, 3, k[0]), vec(rec, 4, r0);
            vec(rec1, 1, b[1]), vec(rec1, 2, w[1]), vec(rec1, 3, k[1]), vec(rec1, 4, r1);
#pragma unroll
            for (int c = 0; c < NC; ++c) v[0][c] = rec[v_at[c]], v[1][c] = rec1[v_at[c]];
            const float beta = rec1[6 * DP], kappa = rec1[6 * DP + 1];
            dots(x0, z), dots(x1, z + NC);
            // all sums in every lane; the outputs of the pair before are summed in the shadow of these exchanges
#pragma unroll
            for (int m = 1; m < S::kLanes; m *= 2) {
#pragma unroll
                for (int i = 0; i < NV; ++i) z[i] += __shfl_xor_sync(0xffffffffu, z[i], m);
            }
            store_outputs();
#pragma unroll
            for (int c = 0; c < NC; ++c) z[NC + c] = z[NC + c] - beta * z[c] + kappa * v[0][c];
            auto update = [&](int j) {
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const f32x2 zz = pair_of(z[j * NC + c], z[j * NC + c]), vv = pair_of(v[j][c], v[j][c]);
#pragma unroll
                    for (int i = 0; i < R2; ++i) st[c][i] = fma2(w[j][i], st[c][i], fma2(k[j][i], vv, mul2(b[j][i], zz)));
                }
            };
            update(0);
            dots(r0, sums);
            if (two) update(1);
            dots(r1, sums + NC);
            held = ch * S::kChunk + t, held_two = two;
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
        for (int i = 0; i < R2; ++i) {
            const int    r   = row0 + 2 * i;
            float*       dst = state + (size_t)(col0 + c) * dim + r;
            const float2 f   = halves(st[c][i]);
            if (col0 + c < dim && r < dim) dst[0] = f.x;
            if (col0 + c < dim && r + 1 < dim) dst[1] = f.y;
        }
    }
}

// Head outputs over their root mean square, times the norm weight and the output gate: a warp takes a head of four tokens
constexpr int kFinishTokens = 4;
template<typename E, int PER>  // PER: dimensions per lane
__global__ void __launch_bounds__(256) delta_finish_kernel(const DeltaKernelParams p)
{
    pdl_wait();
    pdl_launch_dependents();
    const DeltaRule& d    = p.d;
    const int        lane = threadIdx.x & 31, t0 = blockIdx.x * kFinishTokens, h = blockIdx.y * 8 + (threadIdx.x >> 5);
    const int        nt   = min(kFinishTokens, p.c.tokens - t0);
    if (blockIdx.y == 0) {
        for (int t = 0; t < nt; ++t) {
            E* out = static_cast<E*>(p.c.out) + (size_t)(t0 + t) * p.c.out_ld;
            for (int n = d.heads * d.dim + threadIdx.x; n < p.c.out_pad; n += 256) out[n] = from_f32<E>(0.f);
        }
    }
    if (h >= d.heads) return;
    float x[kFinishTokens][PER], g[kFinishTokens][PER], nw[PER];
#pragma unroll
    for (int e = 0; e < PER; ++e) nw[e] = lane + 32 * e < d.dim ? d.norm[h * d.dim + lane + 32 * e] : 0.f;
#pragma unroll
    for (int t = 0; t < kFinishTokens; ++t) {
        const float* o   = p.o + ((size_t)(t0 + t) * d.heads + h) * d.dim;
        const E*     row = static_cast<const E*>(p.c.proj) + (size_t)(t0 + t) * p.c.proj_ld + d.g_col + h * d.dim;
#pragma unroll
        for (int e = 0; e < PER; ++e) {
            const int  c  = lane + 32 * e;
            const bool on = t < nt && c < d.dim;
            x[t][e] = on ? o[c] : 0.f, g[t][e] = on ? to_f32(row[c]) : 0.f;
        }
    }
#pragma unroll
    for (int t = 0; t < kFinishTokens; ++t) {
        float sq = 0.f;
#pragma unroll
        for (int e = 0; e < PER; ++e) sq += x[t][e] * x[t][e];
        const float inv = 1.f / sqrtf(warp_sum(sq) / (float)d.dim + d.norm_eps);
        if (t >= nt) break;
        E* out = static_cast<E*>(p.c.out) + (size_t)(t0 + t) * p.c.out_ld + h * d.dim;
#pragma unroll
        for (int e = 0; e < PER; ++e) {
            if (lane + 32 * e < d.dim) out[lane + 32 * e] = from_f32<E>(x[t][e] * inv * nw[e] * sigmoid_f32(g[t][e]));
        }
    }
}

template<typename E>
cudaError_t finish_launch(const DeltaKernelParams& p, cudaStream_t st)
{
    const dim3 grid((p.c.tokens + kFinishTokens - 1) / kFinishTokens, (p.d.heads + 7) / 8);
    if (p.d.dim <= 32) return launch_kernel(delta_finish_kernel<E, 1>, grid, dim3(256), 0, st, p.c.pdl, p);
    if (p.d.dim <= 64) return launch_kernel(delta_finish_kernel<E, 2>, grid, dim3(256), 0, st, p.c.pdl, p);
    if (p.d.dim <= 128) return launch_kernel(delta_finish_kernel<E, 4>, grid, dim3(256), 0, st, p.c.pdl, p);
    return launch_kernel(delta_finish_kernel<E, 8>, grid, dim3(256), 0, st, p.c.pdl, p);
}

// One new token per sequence, one CTA per (head, sequence): decay projection, step, head norm and gate in one kernel.
// Lanes share a column of S as in the scan; the state passes through registers once, and its reads are under way before
// anything else is known.
template<int DP>
struct StepShape {
    static constexpr int  kThreads = 256, kLanes = DP / 8, kColumns = kThreads / kLanes;
    static constexpr int  kPasses = (DP + kColumns - 1) / kColumns;  // columns per thread
    static constexpr bool kHeld   = kPasses <= 8;                    // all of them in registers from the start
    static constexpr int  kPer    = kThreads / DP;                   // threads that share a channel's decay projection
};

template<typename E, int DP>
__global__ void __launch_bounds__(256, DP <= 64 ? 4 : 1) delta_step_kernel(const DeltaKernelParams p)
{
    using S = StepShape<DP>;
    constexpr int kVec = 16 / sizeof(E);
    __shared__ __align__(16) float u[DP], b[DP], w[DP], k[DP], r[DP];
    __shared__ float v[DP], y[DP], red[8];
    const DeltaRule& d    = p.d;
    const int        h    = blockIdx.x, dim = d.dim, n = h * dim;
    const int        tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const SeqSpan    s    = p.c.spans[blockIdx.y];
    const int        part = tid % S::kLanes, lc = tid / S::kLanes;
    float*           state = reinterpret_cast<float*>(s.slab + d.state_off) + (size_t)h * dim * dim;
    const bool       quad = dim % 4 == 0, old = s.live && s.history > 0;
    float            st[S::kHeld ? S::kPasses : 1][8];
    auto load = [&](int pass, float (&x)[8]) {
        const int col = pass * S::kColumns + lc;
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            const int    r0  = q * (DP / 2) + 4 * part;
            const float* src = state + (size_t)col * dim + r0;
            if (old && col < dim && quad && r0 < dim) {
                const float4 f = *reinterpret_cast<const float4*>(src);
                x[4 * q] = f.x, x[4 * q + 1] = f.y, x[4 * q + 2] = f.z, x[4 * q + 3] = f.w;
            }
            else {
#pragma unroll
                for (int e = 0; e < 4; ++e) x[4 * q + e] = old && col < dim && r0 + e < dim ? src[e] : 0.f;
            }
        }
    };
    // written by this layer's kernel of an earlier step: nothing of this step touches it before
    if (S::kHeld) {
#pragma unroll
        for (int i = 0; i < S::kPasses; ++i) load(i, st[i]);
    }
    // constants of this thread's channel
    const int  c  = tid / S::kPer, sub = tid % S::kPer;
    const bool on = c < dim;
    uint4      w2[4];
    const E*   w2_row = static_cast<const E*>(d.w2) + (size_t)(n + (on ? c : 0)) * d.w2_ld;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = (sub + i * S::kPer) * kVec;
        w2[i]       = m < d.rank ? *reinterpret_cast<const uint4*>(w2_row + m) : make_uint4(0, 0, 0, 0);
    }
    const float w0 = on ? d.w0[n + c] : 0.f, ab = on ? d.a_bias[n + c] : 0.f, nw = tid < dim ? d.norm[n + tid] : 0.f;
    pdl_wait();
    pdl_launch_dependents();
    if (!s.live) return;
    const E*    row = static_cast<const E*>(p.c.proj) + (size_t)s.tok0 * p.c.proj_ld;
    const float kc = on ? to_f32(row[d.k_col + n + c]) : 0.f, rc = on ? to_f32(row[d.r_col + n + c]) : 0.f;
    const float vc = on ? to_f32(row[d.v_col + n + c]) : 0.f, ac = on ? to_f32(row[d.a_col + n + c]) : 0.f;
    const float gate = tid < dim ? to_f32(row[d.g_col + n + tid]) : 0.f;
    // ---- decay pre-activation: w2 . tanh(w1 h)
    const bool aligned = (reinterpret_cast<uintptr_t>(row + d.w1_col) & 15) == 0;
    float      x       = 0.f;
    for (int i = 0;; ++i) {
        const int m = (sub + i * S::kPer) * kVec;
        if (m >= d.rank) break;
        const uint4 a = i == 0 ? w2[0] : i == 1 ? w2[1] : i == 2 ? w2[2] : i == 3 ? w2[3] : *reinterpret_cast<const uint4*>(w2_row + m);
        const E*    wa = reinterpret_cast<const E*>(&a);
        const E*    xa = row + d.w1_col + m;
        if (m + kVec <= d.rank && aligned) {
            const uint4 c16 = *reinterpret_cast<const uint4*>(xa);
            const E*    xe  = reinterpret_cast<const E*>(&c16);
#pragma unroll
            for (int e = 0; e < kVec; ++e) x = fmaf(to_f32(wa[e]), to_f32(xe[e]), x);
        }
        else {
#pragma unroll
            for (int e = 0; e < kVec; ++e) {
                if (m + e < d.rank) x = fmaf(to_f32(wa[e]), to_f32(xa[e]), x);
            }
        }
    }
    // the threads of a channel are neighbours; up to 16 of them
#pragma unroll
    for (int m = 1; m < S::kPer; m *= 2) x += __shfl_xor_sync(0xffffffffu, x, m);
    const float ksq = warp_sum(sub == 0 ? kc * kc : 0.f);
    if (lane == 0) red[warp] = ksq;
    __syncthreads();
    if (sub == 0 && c < DP) {
        float total = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) total += red[i];
        const float uc = kc / sqrtf(total + d.unit_eps);
        u[c] = uc, b[c] = sigmoid_f32(ac + ab) * uc, w[c] = on ? expf(-d.decay_scale * sigmoid_f32(x + w0)) : 0.f;
        k[c] = kc, r[c] = rc, v[c] = vc;
    }
    __syncthreads();
    // ---- the step
    auto vec = [&](const float* a, float (&f)[8]) {
        const float4 lo = *reinterpret_cast<const float4*>(a + 4 * part), hi = *reinterpret_cast<const float4*>(a + DP / 2 + 4 * part);
        f[0] = lo.x, f[1] = lo.y, f[2] = lo.z, f[3] = lo.w, f[4] = hi.x, f[5] = hi.y, f[6] = hi.z, f[7] = hi.w;
    };
    float uu[8], bb[8], ww[8], kk[8], rr[8];
    vec(u, uu), vec(b, bb), vec(w, ww), vec(k, kk), vec(r, rr);
    float sq = 0.f;
#pragma unroll
    for (int pass = 0; pass < S::kPasses; ++pass) {
        float now[8];
        if (S::kHeld) {
#pragma unroll
            for (int i = 0; i < 8; ++i) now[i] = st[S::kHeld ? pass : 0][i];
        }
        else {
            load(pass, now);
        }
        const int   col = pass * S::kColumns + lc;
        const float vj  = col < DP ? v[min(col, DP - 1)] : 0.f;
        float       z = 0.f, o = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) z = fmaf(uu[i], now[i], z);
#pragma unroll
        for (int m = S::kLanes / 2; m >= 1; m >>= 1) z += __shfl_xor_sync(0xffffffffu, z, m);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            now[i] = fmaf(ww[i], now[i], fmaf(kk[i], vj, -bb[i] * z));
            o      = fmaf(rr[i], now[i], o);
        }
#pragma unroll
        for (int m = S::kLanes / 2; m >= 1; m >>= 1) o += __shfl_xor_sync(0xffffffffu, o, m);
        if (col < dim) {
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                const int r0  = q * (DP / 2) + 4 * part;
                float*    dst = state + (size_t)col * dim + r0;
                if (quad && r0 < dim) {
                    *reinterpret_cast<float4*>(dst) = make_float4(now[4 * q], now[4 * q + 1], now[4 * q + 2], now[4 * q + 3]);
                }
                else {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        if (r0 + e < dim) dst[e] = now[4 * q + e];
                    }
                }
            }
            if (part == 0) {
                y[col] = o;
                sq += o * o;
            }
        }
    }
    sq = warp_sum(sq);
    __syncthreads();  // the first use of red is over for everybody
    if (lane == 0) red[warp] = sq;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) total += red[i];
    const float inv = 1.f / sqrtf(total / (float)dim + d.norm_eps);
    E*          out = static_cast<E*>(p.c.out) + (size_t)s.tok0 * p.c.out_ld;
    if (tid < dim) out[n + tid] = from_f32<E>(y[tid] * inv * nw * sigmoid_f32(gate));
    if (h == d.heads - 1) {
        for (int i = d.heads * dim + tid; i < p.c.out_pad; i += S::kThreads) out[i] = from_f32<E>(0.f);
    }
}

template<typename E, int DP>
cudaError_t scan_launch(const DeltaKernelParams& p, cudaStream_t st)
{
    using S       = ScanShape<DP>;
    cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::kSmem);
    if (e != cudaSuccess) return e;
    e = launch_kernel(delta_gates_kernel<E, DP>, dim3((p.c.max_n + 1) / 2, (p.d.heads + 3) / 4, p.c.batch), dim3(128), 0, st, p.c.pdl, p);
    if (e != cudaSuccess) return e;
    const dim3 grid((p.d.dim + S::kColumns - 1) / S::kColumns, p.d.heads, p.c.batch);
    return launch_kernel(delta_scan_kernel<DP>, grid, dim3(S::kThreads), S::kSmem, st, p.c.pdl, p);
}

int padded_dim(int dim)
{
    int dp = 16;
    while (dp < dim) dp *= 2;
    return dp;
}

int scan_dim(int dim)
{
    return padded_dim(dim) < 32 ? 32 : padded_dim(dim);
}

template<typename E>
cudaError_t scan_dispatch(const DeltaKernelParams& p, cudaStream_t st)
{
    switch (scan_dim(p.d.dim)) {
        case 32: return scan_launch<E, 32>(p, st);
        case 64: return scan_launch<E, 64>(p, st);
        case 128: return scan_launch<E, 128>(p, st);
        default: return scan_launch<E, 256>(p, st);
    }
}

template<typename E>
cudaError_t step_dispatch(const DeltaKernelParams& p, cudaStream_t st)
{
    const dim3 grid(p.d.heads, p.c.batch), block(256);
    switch (padded_dim(p.d.dim)) {
        case 16: return launch_kernel(delta_step_kernel<E, 16>, grid, block, 0, st, p.c.pdl, p);
        case 32: return launch_kernel(delta_step_kernel<E, 32>, grid, block, 0, st, p.c.pdl, p);
        case 64: return launch_kernel(delta_step_kernel<E, 64>, grid, block, 0, st, p.c.pdl, p);
        case 128: return launch_kernel(delta_step_kernel<E, 128>, grid, block, 0, st, p.c.pdl, p);
        default: return launch_kernel(delta_step_kernel<E, 256>, grid, block, 0, st, p.c.pdl, p);
    }
}

bool valid(const DeltaRule& d, const MixerCall& c)
{
    return d.heads > 0 && d.heads <= 65535 && d.dim > 0 && d.dim <= kMaxDim && d.rank > 0 && c.batch > 0 && c.batch <= 65535 && c.tokens > 0;
}

}  // namespace

// decay pre-activations, later the outputs, to a multiple of four floats; behind them the records
size_t delta_rule_scratch_floats(const DeltaRule& d)
{
    return (size_t)(d.heads * d.dim + 3) / 4 * 4 + (size_t)d.heads * (6 * scan_dim(d.dim) + 4);
}

int delta_rule_prefill(tm_handle* h, const DeltaRule& d, const MixerCall& c, float* scratch, cudaStream_t st)
{
    if (!valid(d, c) || !scratch) return TM_ERR_UNSUPPORTED;
    const size_t esz = c.f32 ? 4 : 2;
    DenseGemm    g;
    g.w = d.w2, g.ldw = d.w2_ld;
    g.x = static_cast<const char*>(c.proj) + d.w1_col * esz, g.ldx = c.proj_ld;
    g.tokens = c.tokens, g.n_out = d.heads * d.dim, g.k = d.rank;
    g.ep.kind = DenseKind::kF32, g.ep.out = scratch, g.ep.out_ld = d.heads * d.dim;
    const int rc = dense_gemm(h, g, c.f32, st, c.pdl);
    if (rc != TM_OK) return rc;
    float* const            records = scratch + (size_t)c.tokens * ((d.heads * d.dim + 3) / 4 * 4);
    const DeltaKernelParams p{d, c, scratch, records, scratch, h->status, kMaxWaitCycles};
    cudaError_t             e = c.f32 ? scan_dispatch<float>(p, st) : scan_dispatch<__nv_bfloat16>(p, st);
    if (e == cudaSuccess) {
        e = c.f32 ? finish_launch<float>(p, st) : finish_launch<__nv_bfloat16>(p, st);
    }
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    h->launches += 3;
    return TM_OK;
}

int delta_rule_decode(tm_handle* h, const DeltaRule& d, const MixerCall& c, cudaStream_t st)
{
    if (!valid(d, c)) return TM_ERR_UNSUPPORTED;
    const DeltaKernelParams p{d, c, nullptr, nullptr, nullptr, h->status, kMaxWaitCycles};
    const cudaError_t       e = c.f32 ? step_dispatch<float>(p, st) : step_dispatch<__nv_bfloat16>(p, st);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    ++h->launches;
    return TM_OK;
}

}  // namespace tmb
