// Decode-step attention over a sliding window with pooled blocks (WindowAttention in mixers.h), bf16: rotation of the new q
// and k, cache append, pooling of a block that the new token completes, attention and output gate in one kernel.
//
// CTA = (split of the visible keys, kv head x block of up to 16 of its query heads, sequence), four warps.  The keys a
// sequence sees are numbered pooled rows first, then tokens up to the one before the new; a warp streams its own blocks
// of 16 keys and values through a private cp.async ring (16-byte chunks swizzled by row) and keeps an online softmax:
//   S[head, key] = Q K^T   mma.m16n8k16, Q fragments in registers, K rows through ldmatrix
//   O[head, d]  += P V     P straight from the score fragments, V rows through ldmatrix.trans
// All query heads of a kv head ride on the same bytes.  The last split adds the new token itself.  Splits meet in scratch;
// the last CTA to arrive merges them in split order (no CTA waits for another).
// Before griddepcontrol.wait a CTA only reads its span and rows cached by earlier steps.
#include "common.cuh"
#include "window_attention.h"
#include "tm_b200.h"

#include <algorithm>

namespace tmb {
namespace {

constexpr int   kWarps = 4, kThreads = kWarps * 32, kKeys = 16, kHeads = 16, kStages = 3, kMaxSplits = 32;
constexpr float kLog2e = 1.4426950408889634f;

struct StepParams {
    WindowAttention a;
    MixerCall       c;
    float           scale_log2, cap_in, cap_log2;
    int             splits, head_blocks;
    float*          scratch;  // [sequence][kv head][head block][split][16 heads]{m, l, o[D]}
    int*            tickets;
};

template<int D>
struct StepLayout {
    static constexpr int kRow   = D * 2;          // bytes of a row in shared memory
    static constexpr int kTile  = kKeys * kRow;   // one K or V block
    static constexpr int kRing  = kStages * 2 * kTile;
    static constexpr int kQ     = kHeads * kRow;
    static constexpr int kState = kWarps * kHeads * (D + 2) * 4;  // the warps' results, over the rings once they are done
    static constexpr int kSmem  = (kWarps * kRing > kState ? kWarps * kRing : kState) + kQ;
};

__device__ __forceinline__ void cp_async16z(uint32_t dst, const void* src, int bytes)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// byte offset of 16-byte chunk `chunk` of row `row`
template<int D>
__device__ __forceinline__ uint32_t sw(int row, int chunk)
{
    return (uint32_t)(row * D * 2 + ((chunk ^ (row & 7)) << 4));
}

template<int D>
__global__ void __launch_bounds__(kThreads) window_step_kernel(const StepParams p)
{
    using L = StepLayout<D>;
    using E = __nv_bfloat16;
    extern __shared__ __align__(128) unsigned char sm[];
    __shared__ float cs[128], sn[128], k_new[D], v_new[D], self_score[kHeads];
    __shared__ float s_m[kHeads][kMaxSplits], s_l[kHeads][kMaxSplits], s_top[kHeads], s_sum[kHeads];
    __shared__ int   s_last;
    const WindowAttention& a    = p.a;
    const int              tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const SeqSpan          sp   = p.c.spans[blockIdx.z];
    const int              g = blockIdx.y / p.head_blocks, hb = blockIdx.y % p.head_blocks;
    const int              group = a.heads / a.kv_heads;
    const int              h0 = g * group + hb * kHeads, heads = min(kHeads, group - hb * kHeads);
    const int              i = sp.history;
    const bool             live = sp.live != 0;
    const Visible          vis = visible_of(i, a.window, a.pool);
    const int              total = live ? vis.blocks + i - vis.first : 0;  // without the new token
    const int              blocks16 = (total + kKeys - 1) / kKeys;
    const int              blk0 = (int)((long long)blockIdx.x * blocks16 / p.splits), blk1 = (int)((long long)(blockIdx.x + 1) * blocks16 / p.splits);
    const E*               k_tok = reinterpret_cast<const E*>(sp.slab + a.k_off) + (size_t)g * a.ring * a.dim;
    const E*               v_tok = reinterpret_cast<const E*>(sp.slab + a.v_off) + (size_t)g * a.ring * a.vdim;
    const E*               k_blk = reinterpret_cast<const E*>(sp.slab + a.pk_off) + (size_t)g * a.pool_rows * a.dim;
    const E*               v_blk = reinterpret_cast<const E*>(sp.slab + a.pv_off) + (size_t)g * a.pool_rows * a.vdim;
    const int              slot0 = vis.first % a.ring;  // the visible tokens span less than a ring
    const uint32_t         sm_b = smem_u32(sm), ring = sm_b + L::kQ + warp * L::kRing;

    auto fetch = [&](int b, int stage) {
        const uint32_t dst = ring + stage * 2 * L::kTile;
        if (b < blk1) {
#pragma unroll
            for (int r = 0; r < kKeys * D / 8 / 32; ++r) {
                const int  c = lane + r * 32, row = c / (D / 8), chunk = c % (D / 8), idx = b * kKeys + row;
                const bool in = idx < total, blk = idx < vis.blocks;
                int        slot = idx;
                if (!blk) {
                    slot = slot0 + idx - vis.blocks;
                    if (slot >= a.ring) slot -= a.ring;
                }
                const bool ok_k = in && chunk * 8 < a.dim, ok_v = in && chunk * 8 < a.vdim;
                cp_async16z(dst + sw<D>(row, chunk), (blk ? k_blk : k_tok) + (ok_k ? (size_t)slot * a.dim + chunk * 8 : 0), ok_k ? 16 : 0);
                cp_async16z(dst + L::kTile + sw<D>(row, chunk), (blk ? v_blk : v_tok) + (ok_v ? (size_t)slot * a.vdim + chunk * 8 : 0), ok_v ? 16 : 0);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // ring rows of earlier steps: no kernel of this step writes what is read here
#pragma unroll
    for (int s = 0; s < kStages; ++s) fetch(blk0 + warp + s * kWarps, s);
    for (int d = tid; d < a.rot_dims / 2; d += kThreads) sincosf((float)i * a.inv_freq[d], &sn[d], &cs[d]);
    pdl_wait();
    pdl_launch_dependents();
    if (!live) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        return;
    }
    __syncthreads();
    const E*   row  = static_cast<const E*>(p.c.proj) + (size_t)sp.tok0 * p.c.proj_ld;
    const bool tail = (int)blockIdx.x == p.splits - 1;  // the split that takes the new token
    // ---- q of this block's heads, rotated, as bf16 rows (zeros beyond the heads and the head size)
    for (int w = tid; w < kHeads * D / 2; w += kThreads) {
        const int hh = w / (D / 2), d = 2 * (w % (D / 2));
        float     x = 0.f, y = 0.f;
        if (hh < heads && d < a.dim) {
            const E* q = row + a.q_col + (h0 + hh) * a.dim + d;
            x = to_f32(q[0]), y = to_f32(q[1]);
            if (d < a.rot_dims) {
                const float c = cs[d / 2], s = sn[d / 2], x2 = x * c - y * s;
                y = y * c + x * s, x = x2;
            }
        }
        *reinterpret_cast<uint32_t*>(sm + sw<D>(hh, d / 8) + (d % 8) * 2) = pack_bf16(x, y);
    }
    if (tail) {
        for (int d = 2 * tid; d < D; d += 2 * kThreads) {
            float x = 0.f, y = 0.f;
            if (d < a.dim) {
                const E* k = row + a.k_col + g * a.dim + d;
                x = to_f32(k[0]), y = to_f32(k[1]);
                if (d < a.rot_dims) {
                    const float c = cs[d / 2], s = sn[d / 2], x2 = x * c - y * s;
                    y = y * c + x * s, x = x2;
                }
            }
            k_new[d] = to_f32(from_f32<E>(x)), k_new[d + 1] = to_f32(from_f32<E>(y));
        }
        for (int d = tid; d < D; d += kThreads) v_new[d] = d < a.vdim ? to_f32(row[a.v_col + g * a.vdim + d]) : 0.f;
    }
    __syncthreads();
    if (tail) {
        for (int hh = warp; hh < heads; hh += kWarps) {
            float s = 0.f;
            for (int d = lane; d < D; d += 32) s = fmaf(to_f32(*reinterpret_cast<const E*>(sm + sw<D>(hh, d / 8) + (d % 8) * 2)), k_new[d], s);
            s = warp_sum(s);
            if (lane == 0) self_score[hh] = s;
        }
        __syncthreads();
    }
    auto score = [&](float s) {  // in units of log2
        return p.cap_log2 > 0.f ? fmaf(-2.f * p.cap_log2, __fdividef(1.f, 1.f + ex2(s * p.cap_in)), p.cap_log2) : s * p.scale_log2;
    };

    // ---- online softmax over this warp's blocks; fragment rows r and r + 8 are heads
    uint32_t q[D / 16][4];
#pragma unroll
    for (int k = 0; k < D / 16; ++k) ldsm4(sm_b + sw<D>(lane & 15, 2 * k + (lane >> 4)), q[k]);
    const int  r = lane >> 2, c2 = 2 * (lane & 3);
    const bool upper = heads > 8;  // the fragments' rows 8..15 hold heads
    float     m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[D / 8][4];
#pragma unroll
    for (int n = 0; n < D / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    if (tail && warp == 0) {
        // starts out with the new token
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            if (r + 8 * e < heads) m[e] = score(self_score[r + 8 * e]), l[e] = (lane & 3) == 0 ? 1.f : 0.f;
        }
#pragma unroll
        for (int n = 0; n < D / 8; ++n) o[n][0] = o[n][2] = v_new[8 * n + c2], o[n][1] = o[n][3] = v_new[8 * n + c2 + 1];
    }
    int stage = 0;
    for (int b = blk0 + warp; b < blk1; b += kWarps) {
        asm volatile("cp.async.wait_group %0;" ::"n"(kStages - 1) : "memory");
        __syncwarp();
        const uint32_t kt = ring + stage * 2 * L::kTile, vt = kt + L::kTile;
        float          s[2][4] = {};
#pragma unroll
        for (int k = 0; k < D / 16; ++k) {
            uint32_t f[4];  // keys 0-7 / d low, keys 0-7 / d high, keys 8-15 / d low, keys 8-15 / d high
            ldsm4(kt + sw<D>((lane & 7) + ((lane >> 4) << 3), 2 * k + ((lane >> 3) & 1)), f);
            mma_bf16(s[0], q[k], f[0], f[1]);
            mma_bf16(s[1], q[k], f[2], f[3]);
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int t = 0; t < 2; ++t) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                if (e >= 2 && !upper) continue;
                const bool in = b * kKeys + 8 * t + c2 + (e & 1) < total;
                s[t][e]       = in ? score(s[t][e]) : -INFINITY;
                mx[e >> 1]    = fmaxf(mx[e >> 1], s[t][e]);
            }
        }
        float alpha[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            alpha[e] = 1.f;
            if (e == 1 && !upper) continue;
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
            const float top = fmaxf(m[e], mx[e]);
            alpha[e]        = ex2(m[e] - top);
            m[e]            = top;
            l[e] *= alpha[e];
        }
#pragma unroll
        for (int t = 0; t < 2; ++t) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                if (e >= 2 && !upper) continue;  // products of zero rows of Q: finite, and read by nobody
                s[t][e] = ex2(s[t][e] - m[e >> 1]);
                l[e >> 1] += s[t][e];
            }
        }
        const uint32_t pf[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
#pragma unroll
        for (int n = 0; n < D / 8; n += 2) {
            uint32_t f[4];  // keys 0-7 / d low, keys 8-15 / d low, keys 0-7 / d high, keys 8-15 / d high
            ldsm4t(vt + sw<D>(lane & 15, n + (lane >> 4)), f);
#pragma unroll
            for (int e = 0; e < 4; ++e) o[n][e] *= alpha[e >> 1], o[n + 1][e] *= alpha[e >> 1];
            mma_bf16(o[n], pf, f[0], f[1]);
            mma_bf16(o[n + 1], pf, f[2], f[3]);
        }
        __syncwarp();
        fetch(b + kStages * kWarps, stage);
        stage = stage + 1 == kStages ? 0 : stage + 1;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // the rings are free: they take the warps' results

    float* st = reinterpret_cast<float*>(sm + L::kQ) + (size_t)warp * kHeads * (D + 2);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        float x = l[e];
        x += __shfl_xor_sync(0xffffffffu, x, 1);
        x += __shfl_xor_sync(0xffffffffu, x, 2);
        float* rec = st + (r + 8 * e) * (D + 2);
        if ((lane & 3) == 0) rec[0] = m[e], rec[1] = x;
#pragma unroll
        for (int n = 0; n < D / 8; ++n) rec[2 + 8 * n + c2] = o[n][2 * e], rec[3 + 8 * n + c2] = o[n][2 * e + 1];
    }
    __syncthreads();
    const float* all   = reinterpret_cast<const float*>(sm + L::kQ);
    const size_t item  = ((size_t)blockIdx.z * a.kv_heads + g) * p.head_blocks + hb;
    float*       recs  = p.scratch + item * p.splits * kHeads * (D + 2);
    // merge of `parts` results per head: factors first (one thread per head and part), then the sums over the parts
    auto factors = [&](const float* src, int parts, bool divide) {
        for (int w = tid; w < heads * parts; w += kThreads) {
            const float* x    = src + ((size_t)(w % parts) * kHeads + w / parts) * (D + 2);
            s_m[w / parts][w % parts] = __ldcg(x), s_l[w / parts][w % parts] = __ldcg(x + 1);
        }
        __syncthreads();
        if (tid < heads) {
            float top = -INFINITY, sum = 0.f;
            for (int w = 0; w < parts; ++w) top = fmaxf(top, s_m[tid][w]);
            for (int w = 0; w < parts; ++w) {
                const float f = top == -INFINITY ? 0.f : ex2(s_m[tid][w] - top);
                sum += f * s_l[tid][w];
                s_m[tid][w] = f;
            }
            const float scale = divide ? sigmoid_f32(to_f32(row[a.g_col + h0 + tid])) / sum : 1.f;
            for (int w = 0; w < parts; ++w) s_m[tid][w] *= scale;
            s_top[tid] = top, s_sum[tid] = sum;
        }
        __syncthreads();
    };
    auto combine = [&](const float* src, int parts, int hh, int d) {
        float y = 0.f;
#pragma unroll 8
        for (int w = 0; w < parts; ++w) y = fmaf(s_m[hh][w], __ldcg(src + ((size_t)w * kHeads + hh) * (D + 2) + 2 + d), y);
        return y;
    };
    auto store = [&](int hh, int d, float y) {
        static_cast<E*>(p.c.out)[(size_t)sp.tok0 * p.c.out_ld + (h0 + hh) * a.vdim + d] = from_f32<E>(y);
    };
    // the warps' results, in shared memory
    for (int w = tid; w < heads * kWarps; w += kThreads) {
        const float* x = all + ((size_t)(w % kWarps) * kHeads + w / kWarps) * (D + 2);
        s_m[w / kWarps][w % kWarps] = x[0], s_l[w / kWarps][w % kWarps] = x[1];
    }
    __syncthreads();
    if (tid < heads) {
        float top = -INFINITY, sum = 0.f;
        for (int w = 0; w < kWarps; ++w) top = fmaxf(top, s_m[tid][w]);
        for (int w = 0; w < kWarps; ++w) {
            const float f = top == -INFINITY ? 0.f : ex2(s_m[tid][w] - top);
            sum += f * s_l[tid][w];
            s_m[tid][w] = f;
        }
        const float scale = p.splits == 1 ? sigmoid_f32(to_f32(row[a.g_col + h0 + tid])) / sum : 1.f;
        for (int w = 0; w < kWarps; ++w) s_m[tid][w] *= scale;
        s_top[tid] = top, s_sum[tid] = sum;
    }
    __syncthreads();
    auto of_warps = [&](int hh, int d) {
        float y = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) y = fmaf(s_m[hh][w], all[((size_t)w * kHeads + hh) * (D + 2) + 2 + d], y);
        return y;
    };
    if (p.splits == 1) {
        for (int w = tid; w < heads * a.vdim; w += kThreads) store(w / a.vdim, w % a.vdim, of_warps(w / a.vdim, w % a.vdim));
    }
    else {
        float* mine = recs + (size_t)blockIdx.x * kHeads * (D + 2);
        for (int w = tid; w < heads * D; w += kThreads) __stcg(mine + (w / D) * (D + 2) + 2 + w % D, of_warps(w / D, w % D));
        if (tid < heads) {
            __stcg(mine + tid * (D + 2), s_top[tid]);
            __stcg(mine + tid * (D + 2) + 1, s_sum[tid]);
        }
        __threadfence();
        __syncthreads();
        if (tid == 0) {
            s_last = atomicAdd(p.tickets + item, 1) == p.splits - 1;
            if (s_last) p.tickets[item] = 0;
        }
        __syncthreads();
        if (s_last) {
            __threadfence();
            factors(recs, p.splits, true);
            for (int w = tid; w < heads * a.vdim; w += kThreads) store(w / a.vdim, w % a.vdim, combine(recs, p.splits, w / a.vdim, w % a.vdim));
        }
    }

    // ---- off the critical path: cache append, the block that the new token completes, padding columns
    if (tail && hb == 0) {
        const int slot = i % a.ring;
        E*        kw   = reinterpret_cast<E*>(sp.slab + a.k_off) + ((size_t)g * a.ring + slot) * a.dim;
        E*        vw   = reinterpret_cast<E*>(sp.slab + a.v_off) + ((size_t)g * a.ring + slot) * a.vdim;
        for (int d = tid; d < a.dim; d += kThreads) kw[d] = from_f32<E>(k_new[d]);
        for (int d = tid; d < a.vdim; d += kThreads) vw[d] = from_f32<E>(v_new[d]);
        const int b = a.pool > 0 ? i / a.pool : 0;
        if (a.pool > 0 && (i + 1) % a.pool == 0 && b < a.pool_rows) {
            const float inv = 1.f / (float)a.pool;
            for (int d = tid; d < a.dim + a.vdim; d += kThreads) {
                const bool is_k = d < a.dim;
                const int  e = is_k ? d : d - a.dim, width = is_k ? a.dim : a.vdim;
                const E*   src = (is_k ? k_tok : v_tok) + e;
                float      sum = 0.f;
                for (int j = b * a.pool; j < i; ++j) sum += to_f32(src[(size_t)(j % a.ring) * width]);
                sum += is_k ? k_new[e] : v_new[e];
                (reinterpret_cast<E*>(sp.slab + (is_k ? a.pk_off : a.pv_off)) + ((size_t)g * a.pool_rows + b) * width)[e] = from_f32<E>(sum * inv);
            }
        }
        if (g == a.kv_heads - 1) {
            E* out = static_cast<E*>(p.c.out) + (size_t)sp.tok0 * p.c.out_ld;
            for (int d = a.heads * a.vdim + tid; d < p.c.out_pad; d += kThreads) out[d] = from_f32<E>(0.f);
        }
    }
}

cudaError_t prepare(int)
{
    cudaError_t e = cudaFuncSetAttribute(window_step_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, StepLayout<64>::kSmem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(window_step_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, StepLayout<128>::kSmem);
    return e;
}
const KernelPreparation g_prepare(prepare);

}  // namespace

bool window_attention_step_supported(const WindowAttention& a, const MixerCall& c)
{
    return !c.f32 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.vdim <= 128 && a.rot_dims / 2 <= 128;
}

int window_attention_step(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st)
{
    StepParams p{a, c};
    p.scale_log2  = a.scale * kLog2e;
    p.cap_log2    = a.softcap * kLog2e;
    p.cap_in      = a.softcap > 0.f ? 2.f * kLog2e * a.scale / a.softcap : 0.f;
    p.head_blocks = (a.heads / a.kv_heads + kHeads - 1) / kHeads;
    const int D   = a.dim <= 64 && a.vdim <= 64 ? 64 : 128;
    // the bound on the visible keys is the host's
    const long long items = (long long)c.batch * a.kv_heads * p.head_blocks;
    const long long keys  = a.window > 0 ? (long long)a.window + (a.pool > 0 ? c.max_context / a.pool : 0) : c.max_context;
    // two CTAs fit an SM; a CTA's set-up and the merge cost as much as hundreds of keys, so sequences are split only to
    // occupy SMs that would idle, each warp with at least two blocks of keys
    const long long most = std::min<long long>(kMaxSplits, std::max(1ll, keys / (kKeys * kWarps * 2)));
    long long splits     = std::min((2ll * h->sm_count + items - 1) / items, most);
    if (items >= h->sm_count) splits = 1;
    splits = std::min(splits, (long long)(h->attn_scratch_bytes / (items * kHeads * (D + 2) * 4)));
    if (splits < 1 || items > (long long)h->attn_counter_ints) splits = 1;
    p.splits  = (int)splits;
    p.scratch = static_cast<float*>(h->attn_scratch);
    p.tickets = h->attn_counters;
    if (a.kv_heads * p.head_blocks > 65535) return TM_ERR_UNSUPPORTED;
    const dim3        grid(p.splits, a.kv_heads * p.head_blocks, c.batch);
    const cudaError_t e = D == 64 ? launch_kernel(window_step_kernel<64>, grid, dim3(kThreads), StepLayout<64>::kSmem, st, c.pdl, p) :
                                    launch_kernel(window_step_kernel<128>, grid, dim3(kThreads), StepLayout<128>::kSmem, st, c.pdl, p);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    ++h->launches;
    return TM_OK;
}

}  // namespace tmb
