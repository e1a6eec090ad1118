// Dense GEMM of the config-driven decoder (gemm_dense.h): bf16 on the tcgen05 tensor core, fp32 on the CUDA cores.
//
// dense_tc_kernel: 128 output columns (UMMA M) x up to 256 tokens (UMMA N) per tile, persistent, one CTA per SM.
//   warp 0    one lane feeds a ring of stages with TMA: a [128 weight rows x 64 k] box and a [tokens x 64 k] box,
//             128-byte swizzle (every CTA loads for itself); weight boxes start before the kernel ahead is complete
//   warp 1    allocates TMEM (two accumulators, so that one tile's epilogue overlaps the next tile's products); one lane
//             issues four K16 MMAs per stage and commits the stage back to the loader
//   warps 2-5 epilogue: lane = output column, so that every token's 32 columns leave in one contiguous store
// Work split (choose_plan): whole tiles dealt out to the CTAs; or, with few tiles (a decode step), the k blocks of all tiles
// cut evenly over the CTAs, so that every SM streams the same number of bytes (stream-K).  A tile with several CTAs: each publishes its fp32 part in scratch, the last one to arrive adds the parts up in CTA order (nobody waits, the
// sum does not depend on the order of arrival) and runs the epilogue.
// Groups (a mixture of experts): the rows of a group are known on the device only, so every CTA makes the tile table itself
// from the groups' offsets; a tile is (group, weight tile, token tile), the rest is the same.
// Every wait is bounded: a barrier that does not complete sets a status bit, the CTA drains its copies and leaves.
#include "gemm_dense.h"
#include "numeric.cuh"
#include "tcgen05.cuh"
#include "tm_b200.h"

#include <algorithm>

namespace tmb {
namespace {

constexpr int kKBlock    = 64;  // k per stage: 128 bytes per row, the swizzle span
constexpr int kThreads   = 6 * 32;
constexpr int kMaxStages = 12;
constexpr int kMaxTokens = 256;  // tokens of one tile
constexpr int kEpiBar    = 1;    // named barrier of the epilogue warps

struct DenseShared {
    uint64_t full[kMaxStages], empty[kMaxStages];
    uint64_t acc_full[2], acc_empty[2];
    uint32_t tmem_base;
    int      dead;
    int      last;
    int      stop;
    float    scale[kMaxTokens];
    float    red[4][kMaxTokens];
};
// behind DenseShared, groups only: first tile of every group, [groups + 1]

template<bool FAST>
__device__ __forceinline__ float activate(const DenseEpilogue& ep, float gate, float up)
{
    return ep.activation == DenseActivation::kGeluTanh ? gelu_tanh_f32<FAST>(gate) * up : clamped_swish_f32<FAST>(gate, up, ep.limit, ep.slope);
}

struct DenseTcParams {
    int           tokens, n_out, k_blocks;
    int           token_tile, token_tiles, tiles;
    int           grid_tiles;  // tiles dealt out as a whole (all of them, or none)
    int           cut_ctas;    // > 0: CTAs that share the k blocks of all tiles evenly
    int           stages, tmem_columns;
    int           x2_tile;     // weight tiles from here on multiply the second operand
    int           column_tiles, half_box;
    DenseGroups   groups;
    float*        scratch;
    int*          tickets;
    unsigned*     status;
    long long     max_wait;
    DenseEpilogue ep;
};

// kResidual: what 16 consecutive tokens of one output column add to and are gated by, as it lies in memory, requested ahead
struct ResidualIn {
    float         r[16];
    __nv_bfloat16 gate[16];
};
__device__ __forceinline__ void residual_load(const DenseEpilogue& ep, int t0, int live, int n, int n_out, ResidualIn& in)
{
    const bool col = n < n_out;
#pragma unroll
    for (int i = 0; i < 16; ++i) in.r[i] = i < live && col ? ep.residual[(size_t)(t0 + i) * ep.residual_ld + n] : 0.f;
    if (ep.gate) {
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            in.gate[i] = i < live && col ? static_cast<const __nv_bfloat16*>(ep.gate)[(size_t)(t0 + i) * ep.gate_ld + n] : __nv_bfloat16();
        }
    }
}
__device__ __forceinline__ void residual_add(const DenseEpilogue& ep, const float (&y)[16], const ResidualIn& in, float bias, int t0, int live, int n, int n_out,
                                             float (&sq)[16])
{
    using E        = __nv_bfloat16;
    const bool col = n < n_out;
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const bool  on = i < live && col;
        const float f  = ep.gate ? __fdividef(ep.mult, 1.f + __expf(-(to_f32(in.gate[i]) + bias))) : 1.f;
        const float r  = on ? in.r[i] + f * y[i] : 0.f;
        sq[i]          = r * r;
        if (on) ep.residual[(size_t)(t0 + i) * ep.residual_ld + n] = r;
        if (on && ep.cast) static_cast<E*>(ep.cast)[(size_t)(t0 + i) * ep.cast_ld + n] = from_f32<E>(r);
    }
}

// What happens to 16 consecutive tokens of one output column (lane = column); `live` = tokens of the 16 that exist
__device__ __forceinline__ void epilogue16(const DenseEpilogue& ep, const float (&y)[16], int t0, int live, int n, int n_out)
{
    using E        = __nv_bfloat16;
    const bool col = n < n_out;
    if (ep.kind == DenseKind::kF32) {
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            if (i < live && col) static_cast<float*>(ep.out)[(size_t)(t0 + i) * ep.out_ld + n] = y[i];
        }
        return;
    }
    if (ep.kind == DenseKind::kInput && n >= ep.split) {
        // even lanes hold gates, odd lanes the matching ups; of two tokens the even lane finishes one, the odd lane the other
        const bool odd = n & 1;
        E*         dst = static_cast<E*>(ep.act) + ((n - ep.split) >> 1);
#pragma unroll
        for (int i = 0; i < 16; i += 2) {
            const float other = __shfl_xor_sync(0xffffffffu, odd ? y[i] : y[i + 1], 1);
            const float gate = odd ? other : y[i], up = odd ? y[i + 1] : other;
            const int   t = i + (odd ? 1 : 0);
            if (t < live && col) dst[(size_t)(t0 + t) * ep.act_ld] = from_f32<E>(activate<true>(ep, gate, up));
        }
        return;
    }
    if (ep.f32_out && n >= ep.f32_from) {
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            if (i < live && col) ep.f32_out[(size_t)(t0 + i) * ep.f32_ld + n - ep.f32_from] = y[i];
        }
        return;
    }
    const bool th = ep.kind == DenseKind::kInput && n >= ep.tanh_lo && n < ep.tanh_hi;
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        if (i < live && col) static_cast<E*>(ep.out)[(size_t)(t0 + i) * ep.out_ld + n] = from_f32<E>(th ? tanhf(y[i]) : y[i]);
    }
}

template<bool GROUPS>
__global__ void __launch_bounds__(kThreads, 1)
dense_tc_kernel(const DenseTcParams p, const __grid_constant__ CUtensorMap w_map, const __grid_constant__ CUtensorMap x_map,
                const __grid_constant__ CUtensorMap x2_map)
{
    extern __shared__ unsigned char smem_dyn[];
    const uint32_t raw  = smem_u32(smem_dyn);
    const uint32_t base = (raw + 1023u) & ~1023u;  // operand tiles on 1024-byte boundaries (the swizzle is a function of the address)
    const int      NT      = p.token_tile;
    const uint32_t w_bytes = kDenseTile * 128;
    const uint32_t stage_b = w_bytes + (uint32_t)NT * 128;
    const int      ST      = p.stages;
    DenseShared*   sh      = reinterpret_cast<DenseShared*>(smem_dyn + (base - raw) + (size_t)ST * stage_b);
    const int      tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

    if (tid == 0) {
        for (int s = 0; s < kMaxStages; ++s) {
            mbar_init(&sh->full[s], 1);
            mbar_init(&sh->empty[s], 1);
        }
        for (int a = 0; a < 2; ++a) {
            mbar_init(&sh->acc_full[a], 1);
            mbar_init(&sh->acc_empty[a], 4);
        }
        sh->dead = 0;
        fence_mbar_init();
    }
    if (warp == 1) tmem_alloc(&sh->tmem_base, p.tmem_columns);
    int* const first_tile = reinterpret_cast<int*>(sh + 1);
    if (GROUPS) {
        pdl_wait();  // the offsets come from a kernel ahead
        pdl_launch_dependents();
        if (warp == 0) {
            int sum = 0;
            for (int g0 = 0; g0 < p.groups.count; g0 += 32) {
                const int g = g0 + lane;
                int       n = g < p.groups.count ? (p.groups.offsets[g + 1] - p.groups.offsets[g] + NT - 1) / NT * p.column_tiles : 0;
                const int own = n;
#pragma unroll
                for (int m = 1; m < 32; m *= 2) {
                    const int x = __shfl_up_sync(0xffffffffu, n, m);
                    if (lane >= m) n += x;
                }
                if (g < p.groups.count) first_tile[g] = sum + n - own;
                sum += __shfl_sync(0xffffffffu, n, 31);
            }
            if (lane == 0) first_tile[p.groups.count] = sum;
        }
    }
    tcgen05_before_sync();
    __syncthreads();
    tcgen05_after_sync();
    const uint32_t tmem = sh->tmem_base;
    const int      tiles = GROUPS ? first_tile[p.groups.count] : p.tiles;
    // CTAs that share the k blocks; with groups at least four k blocks each, as the host cannot tell how many there are
    const int cut_ctas = GROUPS && p.cut_ctas > 0 ? max(1, min(p.cut_ctas, (int)min((long long)tiles * p.k_blocks / 4, 1ll << 20))) : p.cut_ctas;
    // tile -> weight tile, first row of its tokens, how many there are, first weight row, token tile (the key of `scale`)
    struct Place {
        int ct, t0, rows, w_row, tt, height;  // height: token columns of the tile's products
    };
    auto place = [&](int tile) {
        Place q;
        if (GROUPS) {
            int lo = 0, hi = p.groups.count;  // first_tile[lo] <= tile < first_tile[hi]
            while (hi - lo > 1) {
                const int mid = (lo + hi) >> 1;
                (first_tile[mid] <= tile ? lo : hi) = mid;
            }
            const int begin = p.groups.offsets[lo], n = p.groups.offsets[lo + 1] - begin, tts = (n + NT - 1) / NT, in = tile - first_tile[lo];
            q.ct = in / tts, q.tt = in - q.ct * tts;
            q.height = ((n + tts - 1) / tts + 15) / 16 * 16;  // the group's tiles are equally high
            q.t0 = begin + q.tt * q.height, q.rows = min(q.height, n - q.tt * q.height), q.w_row = lo * p.n_out + q.ct * kDenseTile;
        }
        else {
            q.ct = tile / p.token_tiles, q.tt = tile - q.ct * p.token_tiles;
            q.t0 = q.tt * NT, q.rows = min(NT, p.tokens - q.t0), q.w_row = q.ct * kDenseTile, q.height = NT;
        }
        return q;
    };

    // segment i of this CTA -> tile and k blocks; false behind the last.  Token tiles vary fastest among tiles, so that
    // the CTAs of a wave share weight tiles and activations in the L2.
    const long long cut_total = (long long)tiles * p.k_blocks;
    auto            cut       = [&](int c) { return (long long)c * cut_total / cut_ctas; };
    auto            segment   = [&](int i, int& tile, int& kb0, int& kb1) {
        if (p.cut_ctas == 0) {
            tile = i * (int)gridDim.x + (int)blockIdx.x, kb0 = 0, kb1 = p.k_blocks;
            return tile < (GROUPS ? tiles : p.grid_tiles);
        }
        if (GROUPS && (int)blockIdx.x >= cut_ctas) return false;
        const long long begin = cut(blockIdx.x), end = cut(blockIdx.x + 1), t = begin / p.k_blocks + i;
        if (t * p.k_blocks >= end) return false;
        tile = (int)t, kb0 = (int)(max(begin, t * p.k_blocks) - t * p.k_blocks), kb1 = (int)(min(end, (t + 1) * p.k_blocks) - t * p.k_blocks);
        return true;
    };

    if (warp == 0) {
        // ===================================================================================== loader
        if (lane == 0) {
            int  issued = 0;
            bool ok = true, waited = false;
            // groups: a low tile's rows come in a box of half the height (one copy either way: their issue rate counts)
            auto low    = [&](const Place& q) { return GROUPS && q.height <= p.half_box; };
            auto load_w = [&](int kb, const Place& q, int s) {
                mbar_arrive_expect_tx(&sh->full[s], low(q) ? w_bytes + (uint32_t)p.half_box * 128 : stage_b);
                tma_load_2d(base + s * stage_b, &w_map, kb * kKBlock, q.w_row, &sh->full[s]);
            };
            auto load_x = [&](int kb, const Place& q, int s) {
                tma_load_2d(base + s * stage_b + w_bytes, low(q) || q.ct >= p.x2_tile ? &x2_map : &x_map, kb * kKBlock, q.t0, &sh->full[s]);
            };
            int tile, kb0, kb1;
            for (int seg = 0; ok && segment(seg, tile, kb0, kb1); ++seg) {
                const Place q = place(tile);
                int       kb = kb0;
                if (!waited) {
                    // weights are written by no kernel: the first boxes go out before the kernel ahead is complete
                    const int pre = min(ST, kb1 - kb0);
                    for (int i = 0; i < pre; ++i) load_w(kb0 + i, q, i);
                    pdl_wait();
                    pdl_launch_dependents();
                    waited = true;
                    for (int i = 0; i < pre; ++i) load_x(kb0 + i, q, i);
                    issued = pre;
                    kb += pre;
                }
                for (; kb < kb1; ++kb, ++issued) {
                    const int s = issued % ST;
                    if (issued >= ST && !mbar_wait(&sh->empty[s], ((issued / ST) - 1) & 1, p.max_wait)) {
                        atomicOr(p.status, kStatusGemmPipeWait);
                        *(volatile int*)&sh->dead = 1;
                        ok = false;
                        break;
                    }
                    load_w(kb, q, s);
                    load_x(kb, q, s);
                }
            }
            if (!waited) {
                pdl_wait();
                pdl_launch_dependents();
            }
            if (!ok) {
                // the CTA leaves early: not before its own copies have landed
                for (int i = max(0, issued - ST); i < issued; ++i) mbar_wait(&sh->full[i % ST], (i / ST) & 1, p.max_wait);
            }
        }
        else {
            pdl_wait();
            pdl_launch_dependents();
        }
    }
    else if (warp == 1) {
        // ===================================================================================== MMA issuer
        pdl_wait();
        pdl_launch_dependents();
        if (lane == 0) {
            uint32_t       idesc = umma_idesc_bf16(kDenseTile, NT);
            int            it = 0, local = 0;
            bool           ok = true;
            int            tile, kb0, kb1;
            for (; ok && segment(local, tile, kb0, kb1); ++local) {
                const int a = local & 1;
                if (GROUPS) idesc = umma_idesc_bf16(kDenseTile, place(tile).height);
                if (local >= 2 && !mbar_wait(&sh->acc_empty[a], ((local >> 1) - 1) & 1, p.max_wait)) ok = false;
                tcgen05_after_sync();
                for (int kb = kb0; kb < kb1 && ok; ++kb, ++it) {
                    const int s = it % ST;
                    if (!mbar_wait(&sh->full[s], (it / ST) & 1, p.max_wait)) {
                        ok = false;
                        break;
                    }
                    tcgen05_after_sync();
                    const uint64_t da = umma_desc_k(base + s * stage_b), db = umma_desc_k(base + s * stage_b + w_bytes);
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        umma_f16_ss(tmem + a * NT, da + (uint64_t)(2 * j), db + (uint64_t)(2 * j), idesc, (kb > kb0 || j) ? 1u : 0u);
                    }
                    umma_commit(&sh->empty[s]);
                }
                if (!ok) {
                    atomicOr(p.status, kStatusGemmPipeWait);
                    *(volatile int*)&sh->dead = 1;
                }
                umma_commit(&sh->acc_full[a]);  // arrives when everything issued so far is complete (also on the give-up path)
            }
        }
    }
    else {
        // ===================================================================================== epilogue
        pdl_wait();
        pdl_launch_dependents();
        const int q    = warp & 3;  // the TMEM lane quarter this warp may read
        const int etid = tid - 64;
        const int col  = q * 32 + lane;
        int       local = 0, scaled_tile = -1;
        bool      ok = true;
        int       tile, kb0, kb1;
        for (; ok && segment(local, tile, kb0, kb1); ++local) {
            const Place at = place(tile);
            const int   ct = at.ct, tt = at.tt, a = local & 1, t0 = at.t0, rows = at.rows;
            const int   n = ct * kDenseTile + col;
            if (p.ep.ssq && scaled_tile != tt) {
                // 1 / rms of every token of the tile, once per token tile
                named_bar_sync(kEpiBar, 128);
                for (int t = etid; t < rows; t += 128) {
                    float ss = 0.f;
                    for (int i = 0; i < p.ep.ssq_parts; ++i) ss += p.ep.ssq[(size_t)i * p.ep.ssq_stride + t0 + t];
                    sh->scale[t] = *p.ep.gain / sqrtf(ss * p.ep.inv_width + p.ep.eps);
                }
                named_bar_sync(kEpiBar, 128);
                scaled_tile = tt;
            }
            const bool  adds = p.ep.kind == DenseKind::kResidual;
            const float bias = adds && p.ep.gate && n < p.n_out ? p.ep.gate_bias[n] : 0.f;
            ResidualIn  in;
            if (adds && kb1 - kb0 == p.k_blocks) residual_load(p.ep, t0, min(16, rows), n, p.n_out, in);
            int okw = 1;
            if (lane == 0) okw = mbar_wait(&sh->acc_full[a], (local >> 1) & 1, p.max_wait) ? 1 : 0;
            okw = __shfl_sync(0xffffffffu, okw, 0);
            if (!okw && lane == 0) {
                atomicOr(p.status, kStatusGemmTmemWait);
                *(volatile int*)&sh->dead = 1;
            }
            // one thread decides for all four warps, which share the barriers below
            named_bar_sync(kEpiBar, 128);
            if (etid == 0) sh->stop = *(volatile int*)&sh->dead;
            named_bar_sync(kEpiBar, 128);
            if (*(volatile int*)&sh->stop) {
                ok = false;
                break;
            }
            tcgen05_after_sync();
            const uint32_t acc    = tmem + ((uint32_t)(q * 32) << 16) + (uint32_t)(a * NT);
            bool           finish = true;
            int            parts = 1, part0 = 0;  // CTAs that share this tile: part0, part0 + 1, ...
            const size_t   slot_floats = (size_t)NT * kDenseTile;
            // slot of a CTA's part of the tile: two per CTA, the second for the tile its range ends in
            auto slot_of = [&](int c) { return p.scratch + (size_t)(2 * c + (cut(c) / p.k_blocks == tile ? 0 : 1)) * slot_floats; };
            if (kb1 - kb0 < p.k_blocks) {
                const long long lo = (long long)tile * p.k_blocks, hi = lo + p.k_blocks - 1;
                part0 = (int)(lo * cut_ctas / cut_total);
                while (cut(part0 + 1) <= lo) ++part0;
                while (cut(part0) > lo) --part0;
                int last = (int)(hi * cut_ctas / cut_total);
                while (cut(last + 1) <= hi) ++last;
                while (cut(last) > hi) --last;
                parts       = last - part0 + 1;
                float* mine = slot_of(blockIdx.x);
                for (int c0 = 0; c0 < rows; c0 += 16) {
                    float v[16];
                    tmem_load16(acc + c0, v);
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        if (c0 + i < rows) __stcg(mine + (size_t)(c0 + i) * kDenseTile + col, v[i]);
                    }
                }
                __threadfence();
                named_bar_sync(kEpiBar, 128);
                if (etid == 0) {
                    int*      ticket = p.tickets + tile;
                    const int before = atomicAdd(ticket, 1);
                    sh->last         = before == parts - 1;
                    if (sh->last) *ticket = 0;
                }
                named_bar_sync(kEpiBar, 128);
                finish = *(volatile int*)&sh->last != 0;
                if (finish) __threadfence();
            }
            if (finish) {
                const bool sums = adds && p.ep.ssq_out;
                if (adds && kb1 - kb0 < p.k_blocks) residual_load(p.ep, t0, min(16, rows), n, p.n_out, in);
                for (int c0 = 0; c0 < rows; c0 += 16) {
                    float     v[16], sq[16];
                    const int live = min(16, rows - c0);
                    if (parts > 1) {
#pragma unroll
                        for (int i = 0; i < 16; ++i) v[i] = 0.f;
                        // four parts on their way at a time (a row beyond `live` is scratch of the same slot)
                        for (int c = part0; c < part0 + parts; c += 4) {
                            float x[4][16];
#pragma unroll
                            for (int j = 0; j < 4; ++j) {
                                const float* src = slot_of(min(c + j, part0 + parts - 1)) + (size_t)c0 * kDenseTile + col;
#pragma unroll
                                for (int i = 0; i < 16; ++i) x[j][i] = __ldcg(src + (size_t)i * kDenseTile);
                            }
#pragma unroll
                            for (int j = 0; j < 4; ++j) {
                                if (c + j >= part0 + parts) break;
#pragma unroll
                                for (int i = 0; i < 16; ++i) v[i] += x[j][i];
                            }
                        }
                    }
                    else {
                        tmem_load16(acc + c0, v);
                    }
                    if (p.ep.ssq) {
#pragma unroll
                        for (int i = 0; i < 16; ++i) v[i] *= i < live ? sh->scale[c0 + i] : 0.f;
                    }
                    if (adds) {
                        ResidualIn next;
                        if (c0 + 16 < rows) residual_load(p.ep, t0 + c0 + 16, min(16, rows - c0 - 16), n, p.n_out, next);
                        residual_add(p.ep, v, in, bias, t0 + c0, live, n, p.n_out, sq);
                        in = next;
                    }
                    else {
                        epilogue16(p.ep, v, t0 + c0, live, n, p.n_out);
                    }
                    if (sums) {
#pragma unroll
                        for (int i = 0; i < 16; ++i) {
                            const float s = warp_sum(sq[i]);
                            if (lane == i) sh->red[q][c0 + i] = s;
                        }
                    }
                }
                if (sums) {
                    named_bar_sync(kEpiBar, 128);
                    for (int t = etid; t < rows; t += 128) {
                        p.ep.ssq_out[(size_t)ct * p.ep.ssq_out_stride + t0 + t] = (sh->red[0][t] + sh->red[1][t]) + (sh->red[2][t] + sh->red[3][t]);
                    }
                    named_bar_sync(kEpiBar, 128);
                }
            }
            tcgen05_before_sync();
            __syncwarp();
            if (lane == 0) mbar_arrive(&sh->acc_empty[a]);
        }
    }

    tcgen05_before_sync();
    __syncthreads();
    if (warp == 1) tmem_free(tmem, p.tmem_columns);
}

// ------------------------------------------------------------------------------------------------ fp32
constexpr int kSimtTile = 64, kSimtK = 16;

__global__ void __launch_bounds__(256) dense_f32_kernel(DenseGemm g)
{
    __shared__ float xs[kSimtK][kSimtTile + 4], ws[kSimtK][kSimtTile + 4];
    pdl_wait();
    pdl_launch_dependents();
    const int n0 = blockIdx.x * kSimtTile;
    int       t0 = blockIdx.y * kSimtTile;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const float* x = static_cast<const float*>(g.x2 && n0 >= g.x2_from ? g.x2 : g.x);
    const float* w = static_cast<const float*>(g.w);
    if (g.groups.count > 0) {
        t0 += g.groups.offsets[blockIdx.z];
        g.tokens = g.groups.offsets[blockIdx.z + 1];
        w += (size_t)blockIdx.z * g.n_out * g.ldw;
        if (t0 >= g.tokens) return;
    }
    float        acc[4][4] = {};
    for (int k0 = 0; k0 < g.k; k0 += kSimtK) {
        for (int i = threadIdx.x; i < kSimtTile * kSimtK; i += 256) {
            const int r = i / kSimtK, kk = i % kSimtK, k = k0 + kk;
            xs[kk][r] = t0 + r < g.tokens && k < g.k ? x[(size_t)(t0 + r) * g.ldx + k] : 0.f;
            ws[kk][r] = n0 + r < g.n_out && k < g.k ? w[(size_t)(n0 + r) * g.ldw + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < kSimtK; ++kk) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = xs[kk][ty * 4 + i], b[i] = ws[kk][tx * 4 + i];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
    const DenseEpilogue& ep = g.ep;
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= g.tokens) continue;
        float scale = 1.f;
        if (ep.ssq) {
            float ss = 0.f;
            for (int p = 0; p < ep.ssq_parts; ++p) ss += ep.ssq[(size_t)p * ep.ssq_stride + t];
            scale = *ep.gain / sqrtf(ss * ep.inv_width + ep.eps);
        }
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= g.n_out) continue;
            const float y = acc[i][j] * scale;
            if (ep.kind == DenseKind::kResidual) {
                const float f = ep.gate ? ep.mult * sigmoid_f32(static_cast<const float*>(ep.gate)[(size_t)t * ep.gate_ld + n] + ep.gate_bias[n]) : 1.f;
                ep.residual[(size_t)t * ep.residual_ld + n] += f * y;
            }
            else if (ep.kind == DenseKind::kInput && n >= ep.split) {
                if ((j & 1) == 0) {
                    const float up = n + 1 < g.n_out ? acc[i][j + 1] * scale : 0.f;
                    static_cast<float*>(ep.act)[(size_t)t * ep.act_ld + ((n - ep.split) >> 1)] = activate<false>(ep, y, up);
                }
            }
            else if (ep.f32_out && n >= ep.f32_from) {
                ep.f32_out[(size_t)t * ep.f32_ld + n - ep.f32_from] = y;
            }
            else {
                const bool th = ep.kind == DenseKind::kInput && n >= ep.tanh_lo && n < ep.tanh_hi;
                static_cast<float*>(ep.out)[(size_t)t * ep.out_ld + n] = th ? tanhf(y) : y;
            }
        }
    }
}

using EncodeTiled = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                 const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiled lookup_encode_tiled()
{
    void*                           fn = nullptr;
    cudaDriverEntryPointQueryResult q{};
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) {
        return nullptr;
    }
    return reinterpret_cast<EncodeTiled>(fn);
}

bool encode_rows(EncodeTiled encode, CUtensorMap* map, const void* ptr, int rows, int k, int ld, int box_rows)
{
    const cuuint64_t dims[2]    = {(cuuint64_t)k, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2]     = {(cuuint32_t)kKBlock, (cuuint32_t)box_rows};
    const cuuint32_t estr[2]    = {1u, 1u};
    return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                  CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE)
           == CUDA_SUCCESS;
}

cudaError_t dense_prepare(int max_smem)
{
    const cudaError_t e = cudaFuncSetAttribute(dense_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem);
    return e == cudaSuccess ? cudaFuncSetAttribute(dense_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem) : e;
}
const KernelPreparation g_prepare(dense_prepare);

struct Plan {
    int  token_tile;
    bool cut;
};
// Tile height and whether the tiles are cut, by a model of the launch's time in microseconds: a k block takes what its
// bytes or its products need, cutting costs the exchange of the parts.
Plan choose_plan(int tokens, int n_out, int k_blocks, int sms)
{
    Plan   best{0, false};
    double best_cost = 1e30;
    const int first = tokens >= kMaxTokens ? kMaxTokens : (tokens + 15) / 16 * 16;
    const int last  = tokens >= kMaxTokens ? 128 : first;
    for (int nt = first; nt >= last; nt -= 16) {
        const long long tiles = (long long)((n_out + kDenseTile - 1) / kDenseTile) * ((tokens + nt - 1) / nt);
        const double    block = std::max(0.4, 0.45 * nt / 256);
        const double    whole = (double)((tiles + sms - 1) / sms) * (k_blocks * block + 1.0);
        const double    cut   = (double)tiles * k_blocks / sms * block + 3.0 + 0.06 * nt;
        if (whole < best_cost - 1e-9) best_cost = whole, best = {nt, false};
        if (tiles < 2 * sms && cut < best_cost - 1e-9) best_cost = cut, best = {nt, true};
    }
    return best;
}

// The same for groups, whose rows are spread in a way the host does not know: tiles twice as high as the average group
// (an uneven spread seldom needs a second tile of the same weights), cut unless there are many.
Plan choose_group_plan(int rows, int groups, int n_out, int sms)
{
    const int       average = (rows + groups - 1) / groups;
    const int       nt      = std::min(kMaxTokens, (2 * average + 15) / 16 * 16);
    const long long tiles   = (long long)((n_out + kDenseTile - 1) / kDenseTile) * std::min(rows, groups + rows / nt);
    return {nt, tiles < 4 * sms};
}

int dense_tc(tm_handle* h, const DenseGemm& g, cudaStream_t st, bool pdl)
{
    static const EncodeTiled encode = lookup_encode_tiled();
    if (!encode) return TM_ERR_CUDA;
    if (g.ldw % 8 || g.ldx % 8 || (reinterpret_cast<uintptr_t>(g.w) & 15) || (reinterpret_cast<uintptr_t>(g.x) & 15)) return TM_ERR_INVALID_ARG;
    if (g.ep.kind == DenseKind::kInput && g.ep.split % kDenseTile) return TM_ERR_INVALID_ARG;
    if (g.x2 && (g.x2_from % kDenseTile || (reinterpret_cast<uintptr_t>(g.x2) & 15))) return TM_ERR_INVALID_ARG;
    if (g.groups.count > kMaxDenseGroups || (g.groups.count > 0 && (g.ep.ssq || g.ep.ssq_out || g.x2))) return TM_ERR_UNSUPPORTED;
    DenseTcParams p{};
    p.tokens       = g.tokens;
    p.n_out        = g.n_out;
    p.k_blocks     = (g.k + kKBlock - 1) / kKBlock;
    const bool grouped = g.groups.count > 0;
    const Plan plan    = grouped ? choose_group_plan(g.tokens, g.groups.count, g.n_out, h->sm_count) : choose_plan(g.tokens, g.n_out, p.k_blocks, h->sm_count);
    p.groups           = g.groups;
    p.x2_tile          = g.x2 ? g.x2_from / kDenseTile : 1 << 30;
    p.column_tiles     = (g.n_out + kDenseTile - 1) / kDenseTile;
    p.half_box         = plan.token_tile / 2 / 16 * 16;
    p.token_tile    = plan.token_tile;
    p.token_tiles   = (g.tokens + p.token_tile - 1) / p.token_tile;
    p.tiles         = (g.n_out + kDenseTile - 1) / kDenseTile * p.token_tiles;
    p.tmem_columns = 32;
    while (p.tmem_columns < 2 * p.token_tile) p.tmem_columns *= 2;
    const size_t stage_b = (size_t)kDenseTile * 128 + (size_t)p.token_tile * 128;
    const size_t shared  = sizeof(DenseShared) + (grouped ? (size_t)(g.groups.count + 1) * sizeof(int) : 0);
    p.stages             = (int)(((size_t)h->max_smem - 1024 - shared) / stage_b);
    if (p.stages > kMaxStages) p.stages = kMaxStages;
    if (p.stages < 2) return TM_ERR_UNSUPPORTED;
    const int sms = h->sm_count;
    // tiles that tickets have to be there for
    const long long most = grouped ? (long long)p.column_tiles * std::min(g.tokens, g.groups.count + g.tokens / p.token_tile) : p.tiles;
    if (plan.cut && most <= (long long)h->counter_ints && (size_t)2 * sms * p.token_tile * kDenseTile * 4 <= h->scratch_bytes) {
        // each CTA gets at least four k blocks
        p.cut_ctas = grouped ? sms : (int)std::min<long long>(sms, std::max<long long>(1, (long long)p.tiles * p.k_blocks / 4));
    }
    p.grid_tiles        = p.cut_ctas > 0 ? 0 : p.tiles;
    const int grid_ctas = p.cut_ctas > 0 ? p.cut_ctas : (int)std::min<long long>(sms, most);
    p.scratch  = static_cast<float*>(h->scratch);
    p.tickets  = h->counters;
    p.status   = h->status;
    p.max_wait = h->gemm_wait_cycles > 0 ? h->gemm_wait_cycles : kMaxWaitCycles;
    p.ep       = g.ep;
    CUtensorMap w_map, x_map, x2_map;
    if (!encode_rows(encode, &w_map, g.w, g.n_out * std::max(1, g.groups.count), g.k, g.ldw, kDenseTile)) return TM_ERR_CUDA;
    if (!encode_rows(encode, &x_map, g.x, g.tokens, g.k, g.ldx, p.token_tile)) return TM_ERR_CUDA;
    // the second operand, or the half-height boxes of the groups
    if (!encode_rows(encode, &x2_map, g.x2 ? g.x2 : g.x, g.tokens, g.k, g.ldx, grouped ? std::max(16, p.half_box) : p.token_tile)) return TM_ERR_CUDA;
    const size_t smem = 1024 + (size_t)p.stages * stage_b + shared;
    const dim3   grid(grid_ctas);
    const cudaError_t e = grouped ? launch_kernel(dense_tc_kernel<true>, grid, dim3(kThreads), smem, st, pdl, p, w_map, x_map, x2_map) :
                                    launch_kernel(dense_tc_kernel<false>, grid, dim3(kThreads), smem, st, pdl, p, w_map, x_map, x2_map);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    ++h->launches;
    return TM_OK;
}

}  // namespace

int dense_gemm(tm_handle* h, const DenseGemm& g, bool f32, cudaStream_t st, bool pdl)
{
    if (!g.w || !g.x || g.tokens <= 0 || g.n_out <= 0 || g.k <= 0 || g.ldw < g.k || g.ldx < g.k) return TM_ERR_INVALID_ARG;
    if (!f32) return dense_tc(h, g, st, pdl);
    if (g.ep.kind == DenseKind::kResidual && (g.ep.cast || g.ep.ssq_out)) return TM_ERR_UNSUPPORTED;
    if (g.x2 && g.x2_from % kSimtTile) return TM_ERR_INVALID_ARG;
    const dim3 grid((g.n_out + kSimtTile - 1) / kSimtTile, (g.tokens + kSimtTile - 1) / kSimtTile, std::max(1, g.groups.count));
    const cudaError_t e = launch_kernel(dense_f32_kernel, grid, dim3(256), 0, st, pdl, g);
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    ++h->launches;
    return TM_OK;
}

}  // namespace tmb

using namespace tmb;

extern "C" int tm_gemm_dense(tm_handle* h, void* out, int out_ld, int out_f32, const void* x, int x_ld, const void* w, int w_ld, int tokens,
                             int n_out, int k, int dtype, void* stream)
{
    if (!h || !out || out_ld < n_out || (dtype != TM_DTYPE_BF16 && dtype != TM_DTYPE_F32)) return TM_ERR_INVALID_ARG;
    if (tokens == 0) return TM_OK;
    DenseGemm g;
    g.w = w, g.x = x, g.ldw = w_ld, g.ldx = x_ld, g.tokens = tokens, g.n_out = n_out, g.k = k;
    g.ep.kind = out_f32 ? DenseKind::kF32 : DenseKind::kStore;
    g.ep.out = out, g.ep.out_ld = out_ld;
    return dense_gemm(h, g, dtype == TM_DTYPE_F32, (cudaStream_t)stream, false);
}
