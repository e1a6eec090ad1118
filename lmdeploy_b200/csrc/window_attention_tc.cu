// Prefill attention over a sliding window with pooled blocks (WindowAttention in mixers.h) on the tcgen05 tensor core: bf16,
// head sizes up to 128 in steps of 8 (shorter rows are filled up with zeros in shared memory).
//
// One CTA = 128 queries of one (sequence, head).  It walks over key tiles of 64 rows: first the pooled rows any of its
// queries sees, then the tokens from the oldest one its first query sees to its last query; both kinds are read in place
// from the slab (a tile of tokens starts on a multiple of 64 and the ring is one of 128 rows, so it never wraps inside).
//   warps 0-3   thread = query row = TMEM lane: copy the tiles (cp.async), read the scores from TMEM, mask, softmax, write
//               the probabilities back to TMEM as the A operand of the second product, finally gate and store the output
//   warp 4      allocates TMEM (S 64, P 32, O up to 128 columns); one lane issues S = Q K^T and O += P V
// With a softcap the scores are bounded, so the exponentials need no running maximum and the accumulator no rescaling
// (kBounded); otherwise the maximum is followed only when it is left behind by more than 2^8.
// Two CTAs are resident per SM: one's softmax overlaps the other's products.  Every barrier wait is bounded.
#include "tcgen05.cuh"
#include "window_attention.h"
#include "tm_b200.h"

namespace tmb {
namespace {

constexpr int   kBM = 128, kBN = 64;  // queries of a CTA, keys of a tile
constexpr int   kRowThreads = 128, kThreads = 160;
constexpr int   kTBlock = kBN * 128, kQBlock = kBM * 128;  // bytes of a 64-wide block of head dimensions
constexpr int   kColS = 0, kColP = 64, kColO = 128, kTmemCols = 256;
constexpr float kLog2e      = 1.4426950408889634f;
constexpr float kMaxBounded = 80.f;  // largest softcap * log2(e) whose exponentials and sums stay far inside fp32 and bf16

struct Bars {
    uint64_t kv_full[2];
    uint64_t s_full, p_full, o_full;
    uint32_t tmem_base;
    int      dead;
};

struct TcParams {
    WindowAttention a;
    MixerCall       c;
    float           scale_log2;  // scale * log2(e); bounded: unused
    float           cap_in;      // 2 * log2(e) * scale / softcap
    float           cap_log2;    // softcap * log2(e)
    unsigned*       status;
    long long       max_wait;
};

__device__ __forceinline__ uint32_t sw_off(int row, int chunk, int block_bytes)
{
    return (uint32_t)((chunk >> 3) * block_bytes + row * 128 + (((chunk & 7) ^ (row & 7)) << 4));
}
__device__ __forceinline__ void cp_async16z(uint32_t dst, const void* src, int bytes)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ float ex2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp(float x)
{
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// DK, DV: head sizes rounded up to 64 or 128
template<int DK, int DV>
struct Layout {
    static constexpr int kQBytes = kBM * DK * 2, kKBytes = kBN * DK * 2, kVBytes = kBN * DV * 2;
    static constexpr int kSmem   = 1024 + kQBytes + 2 * (kKBytes + kVBytes) + 128;
};

template<int DK, int DV, bool kBounded>
__global__ void __launch_bounds__(kThreads, 2) window_attention_tc_kernel(const TcParams p)
{
    using L = Layout<DK, DV>;
    using E = __nv_bfloat16;
    extern __shared__ unsigned char smem_dyn[];
    pdl_wait();
    pdl_launch_dependents();
    const WindowAttention& a   = p.a;
    const int              tid = threadIdx.x, warp = tid >> 5;
    const SeqSpan          sp = p.c.spans[blockIdx.z];
    const int              h = blockIdx.y, g = h / (a.heads / a.kv_heads);
    const int              q0 = (gridDim.x - 1 - blockIdx.x) * kBM;  // the longest (latest) query tiles first
    if (!sp.live || q0 >= sp.n) return;                               // the whole CTA, before anything is set up
    const int     rows = min(kBM, sp.n - q0), pos0 = sp.history + q0, pos1 = pos0 + rows - 1;
    const Visible v0 = visible_of(pos0, a.window, a.pool), v1 = visible_of(pos1, a.window, a.pool);
    const int     blk_tiles = (v1.blocks + kBN - 1) / kBN;
    const int     tok_base  = v0.first / kBN * kBN;
    const int     n_tiles   = blk_tiles + (pos1 - tok_base) / kBN + 1;

    const uint32_t raw  = smem_u32(smem_dyn);
    const uint32_t base = (raw + 1023u) & ~1023u;
    const uint32_t kv_s = base + L::kQBytes;  // [buf][k | v]
    Bars*          bars = reinterpret_cast<Bars*>(smem_dyn + (base - raw) + L::kQBytes + 2 * (L::kKBytes + L::kVBytes));
    if (tid == 0) {
        mbar_init(&bars->kv_full[0], kRowThreads);
        mbar_init(&bars->kv_full[1], kRowThreads);
        mbar_init(&bars->s_full, 1);
        mbar_init(&bars->p_full, kRowThreads);
        mbar_init(&bars->o_full, 1);
        bars->dead = 0;
        fence_mbar_init();
    }
    if (warp == 4) tmem_alloc(&bars->tmem_base, kTmemCols);
    tcgen05_before_sync();
    __syncthreads();
    tcgen05_after_sync();
    const uint32_t tmem = bars->tmem_base;

    if (warp < 4) {
        // ============================================================ copies, softmax, output: thread = query row
        const E* k_tok = reinterpret_cast<const E*>(sp.slab + a.k_off) + (size_t)g * a.ring * a.dim;
        const E* v_tok = reinterpret_cast<const E*>(sp.slab + a.v_off) + (size_t)g * a.ring * a.vdim;
        const E* k_blk = reinterpret_cast<const E*>(sp.slab + a.pk_off) + (size_t)g * a.pool_rows * a.dim;
        const E* v_blk = reinterpret_cast<const E*>(sp.slab + a.pv_off) + (size_t)g * a.pool_rows * a.vdim;
        auto load_tile = [&](int t, int buf) {
            const bool pooled = t < blk_tiles;
            const int  key0   = pooled ? t * kBN : tok_base + (t - blk_tiles) * kBN;
            const int  count  = min(kBN, (pooled ? v1.blocks : pos1 + 1) - key0);
            const int  slot   = pooled ? key0 : key0 % a.ring;
            const E *  k_src = (pooled ? k_blk : k_tok) + (size_t)slot * a.dim, *v_src = (pooled ? v_blk : v_tok) + (size_t)slot * a.vdim;
            const uint32_t dst = kv_s + buf * (L::kKBytes + L::kVBytes);
#pragma unroll
            for (int r = 0; r < kBN * DK / 8 / kRowThreads; ++r) {
                const int  c = tid + r * kRowThreads, row = c / (DK / 8), chunk = c % (DK / 8);
                const bool ok = row < count && chunk * 8 < a.dim;
                cp_async16z(dst + sw_off(row, chunk, kTBlock), k_src + (ok ? (size_t)row * a.dim + chunk * 8 : 0), ok ? 16 : 0);
            }
#pragma unroll
            for (int r = 0; r < kBN * DV / 8 / kRowThreads; ++r) {
                const int  c = tid + r * kRowThreads, row = c / (DV / 8), chunk = c % (DV / 8);
                const bool ok = row < count && chunk * 8 < a.vdim;
                cp_async16z(dst + L::kKBytes + sw_off(row, chunk, kTBlock), v_src + (ok ? (size_t)row * a.vdim + chunk * 8 : 0), ok ? 16 : 0);
            }
        };
        {
            const E* qsrc = static_cast<const E*>(p.c.proj) + (size_t)(sp.tok0 + q0) * p.c.proj_ld + a.q_col + h * a.dim;
#pragma unroll
            for (int r = 0; r < kBM * DK / 8 / kRowThreads; ++r) {
                const int  c = tid + r * kRowThreads, row = c / (DK / 8), chunk = c % (DK / 8);
                const bool ok = row < rows && chunk * 8 < a.dim;
                cp_async16z(base + sw_off(row, chunk, kQBlock), qsrc + (ok ? (size_t)row * p.c.proj_ld + chunk * 8 : 0), ok ? 16 : 0);
            }
        }
        load_tile(0, 0);
        asm volatile("cp.async.commit_group;" ::: "memory");

        const bool     live  = tid < rows;
        const int      mine  = pos0 + tid;
        const Visible  vis   = live ? visible_of(mine, a.window, a.pool) : Visible{1 << 30, 0};
        const int      limit = live ? mine : -1;
        const uint32_t lane  = tmem + ((uint32_t)(warp * 32) << 16);
        float          m_used = -INFINITY, l = 0.f;
        bool           dead = false;
        for (int t = 0; t < n_tiles; ++t) {
            const int buf = t & 1;
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            fence_async_shared();  // this thread's copies become visible to the tensor core's reads
            mbar_arrive(&bars->kv_full[buf]);
            // uniform across the warp: the TMEM loads and stores below are warp-wide instructions
            if (!__all_sync(0xffffffffu, mbar_wait(&bars->s_full, t & 1, p.max_wait))) {
                atomicOr(p.status, kStatusGemmPipeWait);
                *(volatile int*)&bars->dead = 1;
                dead = true;
                break;
            }
            tcgen05_after_sync();
            // S of this tile is complete, so every product on the tile before it is too: its buffers are free
            if (t + 1 < n_tiles) load_tile(t + 1, buf ^ 1);
            asm volatile("cp.async.commit_group;" ::: "memory");

            uint32_t s0[32], s1[32];
            tmem_load32(lane + kColS, s0);
            tmem_load32(lane + kColS + 32, s1);
            // keys of the tile this row sees: [lo, hi) of its 64.  Only tiles at an edge mask anything (same for the CTA).
            const bool pooled = t < blk_tiles;
            const int  key0   = pooled ? t * kBN : tok_base + (t - blk_tiles) * kBN;
            const int  lo = pooled ? 0 : vis.first - key0, hi = pooled ? vis.blocks - key0 : limit + 1 - key0;
            const bool edge = pooled ? key0 + kBN > v0.blocks : key0 + kBN - 1 > pos0 || key0 < v1.first;
            const bool mask = edge || rows < kBM;
            float      sum  = 0.f;
            uint32_t   pr[32];
            if (kBounded) {
                // tanh(x) = 1 - 2 / (1 + e^2x): p = 2^(cap log2(e) tanh(scale s / cap))
                auto weight = [&](uint32_t s) {
                    return ex2(fmaf(-2.f * p.cap_log2, rcp(1.f + ex2(__uint_as_float(s) * p.cap_in)), p.cap_log2));
                };
                if (mask) {
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        const float w0 = 2 * i >= lo && 2 * i < hi ? weight(s0[2 * i]) : 0.f;
                        const float w1 = 2 * i + 1 >= lo && 2 * i + 1 < hi ? weight(s0[2 * i + 1]) : 0.f;
                        const float w2 = 2 * i + 32 >= lo && 2 * i + 32 < hi ? weight(s1[2 * i]) : 0.f;
                        const float w3 = 2 * i + 33 >= lo && 2 * i + 33 < hi ? weight(s1[2 * i + 1]) : 0.f;
                        sum += (w0 + w1) + (w2 + w3);
                        pr[i] = pack_bf16(w0, w1), pr[16 + i] = pack_bf16(w2, w3);
                    }
                }
                else {
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        const float w0 = weight(s0[2 * i]), w1 = weight(s0[2 * i + 1]), w2 = weight(s1[2 * i]), w3 = weight(s1[2 * i + 1]);
                        sum += (w0 + w1) + (w2 + w3);
                        pr[i] = pack_bf16(w0, w1), pr[16 + i] = pack_bf16(w2, w3);
                    }
                }
                l += sum;
            }
            else {
                if (p.cap_log2 > 0.f) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        s0[i] = __float_as_uint(fmaf(-2.f * p.cap_log2, rcp(1.f + ex2(__uint_as_float(s0[i]) * p.cap_in)), p.cap_log2));
                        s1[i] = __float_as_uint(fmaf(-2.f * p.cap_log2, rcp(1.f + ex2(__uint_as_float(s1[i]) * p.cap_in)), p.cap_log2));
                    }
                }
                else {
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        s0[i] = __float_as_uint(__uint_as_float(s0[i]) * p.scale_log2);
                        s1[i] = __float_as_uint(__uint_as_float(s1[i]) * p.scale_log2);
                    }
                }
                if (mask) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        if (i < lo || i >= hi) s0[i] = 0xff800000u;  // -inf
                        if (i + 32 < lo || i + 32 >= hi) s1[i] = 0xff800000u;
                    }
                }
                float mx = -INFINITY;
#pragma unroll
                for (int i = 0; i < 32; ++i) mx = fmaxf(mx, fmaxf(__uint_as_float(s0[i]), __uint_as_float(s1[i])));
                float alpha = 1.f;
                if (mx > m_used + 8.f) {
                    alpha  = ex2(m_used - mx);  // 0 where nothing was seen before
                    m_used = mx;
                }
                const float nm = m_used == -INFINITY ? 0.f : -m_used;
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float w0 = ex2(__uint_as_float(s0[2 * i]) + nm), w1 = ex2(__uint_as_float(s0[2 * i + 1]) + nm);
                    const float w2 = ex2(__uint_as_float(s1[2 * i]) + nm), w3 = ex2(__uint_as_float(s1[2 * i + 1]) + nm);
                    sum += (w0 + w1) + (w2 + w3);
                    pr[i] = pack_bf16(w0, w1), pr[16 + i] = pack_bf16(w2, w3);
                }
                l = l * alpha + sum;
                if (t > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll 1
                    for (int c = 0; c < DV / 32; ++c) {
                        uint32_t o[32];
                        tmem_load32(lane + kColO + 32 * c, o);
#pragma unroll
                        for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                        tmem_store32(lane + kColO + 32 * c, o);
                    }
                }
            }
            tmem_store32(lane + kColP, pr);
            tmem_store_wait();
            tcgen05_before_sync();
            mbar_arrive(&bars->p_full);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        if (!dead && !__all_sync(0xffffffffu, mbar_wait(&bars->o_full, 0, p.max_wait))) {
            atomicOr(p.status, kStatusGemmTmemWait);
            dead = true;
        }
        tcgen05_after_sync();
        if (!dead && *(volatile int*)&bars->dead == 0) {
            const size_t t   = (size_t)(sp.tok0 + q0 + tid);
            float        inv = 0.f;
            if (live) inv = sigmoid_f32(to_f32(static_cast<const E*>(p.c.proj)[t * p.c.proj_ld + a.g_col + h])) / l;
            E* out = static_cast<E*>(p.c.out) + t * p.c.out_ld;
#pragma unroll 1
            for (int c = 0; c < DV / 32; ++c) {
                uint32_t o[32];
                tmem_load32(lane + kColO + 32 * c, o);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    if (!live || 32 * c + 8 * i >= a.vdim) continue;
                    uint4 w;
                    w.x = pack_bf16(__uint_as_float(o[8 * i]) * inv, __uint_as_float(o[8 * i + 1]) * inv);
                    w.y = pack_bf16(__uint_as_float(o[8 * i + 2]) * inv, __uint_as_float(o[8 * i + 3]) * inv);
                    w.z = pack_bf16(__uint_as_float(o[8 * i + 4]) * inv, __uint_as_float(o[8 * i + 5]) * inv);
                    w.w = pack_bf16(__uint_as_float(o[8 * i + 6]) * inv, __uint_as_float(o[8 * i + 7]) * inv);
                    *reinterpret_cast<uint4*>(out + h * a.vdim + 32 * c + 8 * i) = w;
                }
            }
            if (live && h == a.heads - 1) {
                for (int d = a.heads * a.vdim; d < p.c.out_pad; ++d) out[d] = from_f32<E>(0.f);
            }
        }
    }
    else if ((tid & 31) == 0) {
        // ============================================================ MMA issuer
        const uint32_t idesc_qk = umma_idesc_bf16(kBM, kBN), idesc_pv = umma_idesc_bf16(kBM, DV, true);
        bool           ok       = true;
        for (int t = 0; t < n_tiles && ok; ++t) {
            const int buf = t & 1;
            if (!mbar_wait(&bars->kv_full[buf], (t >> 1) & 1, p.max_wait)) {
                ok = false;
                break;
            }
            tcgen05_after_sync();
            const uint32_t k_addr = kv_s + buf * (L::kKBytes + L::kVBytes), v_addr = k_addr + L::kKBytes;
#pragma unroll
            for (int blk = 0; blk < DK / 64; ++blk) {
                const uint64_t dq = umma_desc_k(base + blk * kQBlock), dk = umma_desc_k(k_addr + blk * kTBlock);
#pragma unroll
                for (int j = 0; j < 4; ++j) umma_f16_ss(tmem + kColS, dq + (uint64_t)(2 * j), dk + (uint64_t)(2 * j), idesc_qk, (blk | j) ? 1u : 0u);
            }
            umma_commit(&bars->s_full);
            if (!mbar_wait(&bars->p_full, t & 1, p.max_wait)) {
                ok = false;
                break;
            }
            tcgen05_after_sync();
            const uint64_t dv = umma_desc_mn(v_addr, kTBlock);
#pragma unroll
            for (int j = 0; j < 4; ++j) umma_f16_ts(tmem + kColO, tmem + kColP + 8 * j, dv + (uint64_t)(128 * j), idesc_pv, (t | j) ? 1u : 0u);
        }
        if (!ok) {
            atomicOr(p.status, kStatusGemmPipeWait);
            *(volatile int*)&bars->dead = 1;
        }
        umma_commit(&bars->o_full);  // arrives when everything issued so far is complete (also on the give-up path)
    }

    tcgen05_before_sync();
    __syncthreads();
    if (warp == 4) tmem_free(tmem, kTmemCols);
}

template<int DK, int DV>
cudaError_t prepare_one()
{
    cudaError_t e = cudaFuncSetAttribute(window_attention_tc_kernel<DK, DV, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, Layout<DK, DV>::kSmem);
    if (e == cudaSuccess) {
        e = cudaFuncSetAttribute(window_attention_tc_kernel<DK, DV, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, Layout<DK, DV>::kSmem);
    }
    return e;
}
cudaError_t prepare(int)
{
    cudaError_t e = prepare_one<64, 64>();
    if (e == cudaSuccess) e = prepare_one<64, 128>();
    if (e == cudaSuccess) e = prepare_one<128, 64>();
    if (e == cudaSuccess) e = prepare_one<128, 128>();
    return e;
}
const KernelPreparation g_prepare(prepare);

template<int DK, int DV>
cudaError_t launch(const TcParams& p, bool bounded, cudaStream_t st)
{
    const dim3 grid((p.c.max_n + kBM - 1) / kBM, p.a.heads, p.c.batch);
    return launch_kernel(bounded ? window_attention_tc_kernel<DK, DV, true> : window_attention_tc_kernel<DK, DV, false>, grid, dim3(kThreads),
                         Layout<DK, DV>::kSmem, st, p.c.pdl, p);
}

}  // namespace

bool window_attention_tc_supported(const WindowAttention& a, const MixerCall& c)
{
    return !c.f32 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.vdim <= 128 && a.ring % kBN == 0 && a.q_col % 8 == 0
           && c.proj_ld % 8 == 0 && c.out_ld % 8 == 0 && a.scale > 0.f && a.heads <= 65535;
}

int window_attention_tc(tm_handle* h, const WindowAttention& a, const MixerCall& c, cudaStream_t st)
{
    TcParams p{a, c};
    p.scale_log2       = a.scale * kLog2e;
    p.cap_log2         = a.softcap * kLog2e;
    p.cap_in           = a.softcap > 0.f ? 2.f * kLog2e * a.scale / a.softcap : 0.f;
    p.status           = h->status;
    p.max_wait         = kMaxWaitCycles;
    const bool bounded = a.softcap > 0.f && p.cap_log2 <= kMaxBounded;
    const bool k64 = a.dim <= 64, v64 = a.vdim <= 64;
    const cudaError_t e = k64 ? (v64 ? launch<64, 64>(p, bounded, st) : launch<64, 128>(p, bounded, st)) :
                                (v64 ? launch<128, 64>(p, bounded, st) : launch<128, 128>(p, bounded, st));
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    ++h->launches;
    return TM_OK;
}

}  // namespace tmb
