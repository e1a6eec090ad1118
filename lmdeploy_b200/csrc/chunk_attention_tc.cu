// Prefill of the chunk attention (ChunkAttention in mixers.h) on the tensor cores: bf16, head sizes up to 128 in steps of 8
// (shorter rows are filled up with zeros in shared memory), up to 64 heads.
//
// The weights of all heads meet for every (query, key) pair, and neither the weights nor the outputs of all heads of a tile
// fit an SM.  So the pass goes through memory, a block of query tiles (128 queries of one sequence) at a time, as many as
// the scratch holds, [tile][head][query][key]:
//   chunk_scores_kernel   CTA = (head, tile): S = Q K^T (tcgen05, accumulator in TMEM twice, so that the next product runs
//                         under this one's epilogue), sigmoid, mask; fp16 weights
//   chunk_mix_kernel      warp = 64 pairs of a query at a time: [heads x heads] times [heads x pairs] by mma.m16n8k16 with
//                         fragments straight from and to memory, in place; the mixed weights are bf16
//   chunk_values_kernel   CTA = (head, tile): O = P V (tcgen05)
// fp16 holds a weight (times a power of two, kWeightScale) to 2^-12, finer than the bf16 operand of the last product, and the
// mixing matrix, whose elements are bf16 weights, exactly unless they are tiny.  Every barrier wait is bounded.
#include "chunk_attention.h"
#include "tcgen05.cuh"
#include "tm_b200.h"

#include <algorithm>

namespace tmb {
namespace {

constexpr int   kBM = 128, kBN = 64;  // queries and keys of a tile
constexpr int   kRowThreads = 128, kThreads = 160;
constexpr int   kTBlock = kBN * 128, kQBlock = kBM * 128;  // bytes of a 64-wide block of a tile's columns
constexpr int   kStages = 3;                               // of the values kernel
constexpr int   kMixSplit = 2;                             // warps that share the keys of a query
constexpr int   kMaxHeads = 64;
constexpr float kLog2e = 1.4426950408889634f;

struct ChunkTcParams {
    ChunkAttention a;
    MixerCall      c;
    int            tile0;    // first query tile of the block
    int            ldk;      // keys of a row in the scratch
    __half*        weights;
    unsigned*      status;
    long long      max_wait;
};

// A query tile: its span, its queries' positions, and the key tiles they see (the first starts at `base`)
struct TileInfo {
    SeqSpan sp;
    int     q0, rows, pos0, pos1, base, n_tiles;
};
__device__ __forceinline__ TileInfo tile_info(const ChunkTcParams& p, int item)
{
    const QueryTile q = p.c.tiles[p.tile0 + item];
    TileInfo        t;
    t.sp   = p.c.spans[q.span];
    t.q0   = q.q0;
    t.rows = min(kBM, t.sp.n - q.q0), t.pos0 = t.sp.history + q.q0, t.pos1 = t.pos0 + t.rows - 1;
    t.base    = chunk_first(t.pos0, p.a.chunk) / kBN * kBN;
    t.n_tiles = (t.pos1 - t.base) / kBN + 1;
    return t;
}

__device__ __forceinline__ uint32_t sw_off(int row, int chunk, int block_bytes)
{
    return (uint32_t)((chunk >> 3) * block_bytes + row * 128 + (((chunk & 7) ^ (row & 7)) << 4));
}
__device__ __forceinline__ void cp_async16z(uint32_t dst, const void* src, int bytes)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ float scaled_sigmoid_log2(float x)  // sigmoid of x / log2(e), times kWeightScale
{
    float e, y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-x));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(fmaf(e, 1.f / kWeightScale, 1.f / kWeightScale)));
    return y;
}
// rows [0, count) of [row][width] at src into a swizzled tile of ROWS rows and D columns, zeros elsewhere
template<int ROWS, int D>
__device__ __forceinline__ void copy_rows(uint32_t dst, int block_bytes, const __nv_bfloat16* src, size_t ld, int count, int width)
{
#pragma unroll
    for (int r = 0; r < ROWS * D / 8 / kRowThreads; ++r) {
        const int  c = threadIdx.x + r * kRowThreads, row = c / (D / 8), chunk = c % (D / 8);
        const bool ok = row < count && chunk * 8 < width;
        cp_async16z(dst + sw_off(row, chunk, block_bytes), src + (ok ? (size_t)row * ld + chunk * 8 : 0), ok ? 16 : 0);
    }
}

// ------------------------------------------------------------------------------------------------ scores -> weights
struct ScoreBars {
    uint64_t kv_full[2], s_full[2];
    uint32_t tmem_base;
};
template<int DK>
struct ScoreLayout {
    static constexpr int kQ = kBM * DK * 2, kK = kBN * DK * 2, kOut = kBM * kBN * 2;
    static constexpr int kSmem = 1024 + kQ + 2 * kK + kOut + 64;
};

template<int DK>
__global__ void __launch_bounds__(kThreads, 2) chunk_scores_kernel(const ChunkTcParams p)
{
    using L = ScoreLayout<DK>;
    using E = __nv_bfloat16;
    extern __shared__ unsigned char smem_dyn[];
    pdl_wait();
    pdl_launch_dependents();
    const ChunkAttention& a = p.a;
    const int             tid = threadIdx.x, warp = tid >> 5, h = blockIdx.x, g = h / (a.heads / a.kv_heads);
    const TileInfo        ti = tile_info(p, blockIdx.y);
    if (!ti.sp.live || ti.rows <= 0) return;
    const uint32_t raw = smem_u32(smem_dyn), base = (raw + 1023u) & ~1023u;
    const uint32_t k_s = base + L::kQ, out_s = k_s + 2 * L::kK;
    ScoreBars*     bars = reinterpret_cast<ScoreBars*>(smem_dyn + (base - raw) + L::kQ + 2 * L::kK + L::kOut);
    if (tid == 0) {
        for (int i = 0; i < 2; ++i) mbar_init(&bars->kv_full[i], kRowThreads), mbar_init(&bars->s_full[i], 1);
        fence_mbar_init();
    }
    if (warp == 4) tmem_alloc(&bars->tmem_base, 2 * kBN);
    tcgen05_before_sync();
    __syncthreads();
    tcgen05_after_sync();
    const uint32_t tmem = bars->tmem_base;

    if (warp < 4) {
        const E* keys = reinterpret_cast<const E*>(ti.sp.slab + a.k_off) + (size_t)g * a.ring * a.dim;
        // a tile of keys starts on a multiple of 64 and the ring is one of 128 rows, so it never wraps inside
        auto load_keys = [&](int t) {
            const int key0 = ti.base + t * kBN;
            copy_rows<kBN, DK>(k_s + (t & 1) * L::kK, kTBlock, keys + (size_t)(key0 % a.ring) * a.dim, a.dim, min(kBN, ti.pos1 + 1 - key0), a.dim);
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        copy_rows<kBM, DK>(base, kQBlock, static_cast<const E*>(p.c.proj) + (size_t)(ti.sp.tok0 + ti.q0) * p.c.proj_ld + a.q_col + h * a.dim, p.c.proj_ld,
                           ti.rows, a.dim);
        load_keys(0);
        if (ti.n_tiles > 1) {
            load_keys(1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        }
        else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        fence_async_shared();  // this thread's copies become visible to the tensor core's reads
        mbar_arrive(&bars->kv_full[0]);

        const bool     live  = tid < ti.rows;
        const int      mine  = ti.pos0 + tid, lo = live ? chunk_first(mine, a.chunk) : 1 << 30;
        const uint32_t lane  = tmem + ((uint32_t)(warp * 32) << 16);
        const float    scale = a.scale * kLog2e, bias = a.bias[h] * kLog2e;
        __half*        out   = p.weights + ((size_t)blockIdx.y * a.heads + h) * kBM * p.ldk;
        bool           dead  = false;
        for (int t = 0; t < ti.n_tiles; ++t) {
            if (t + 1 < ti.n_tiles) {
                asm volatile("cp.async.wait_group 0;" ::: "memory");
                fence_async_shared();
                tcgen05_before_sync();  // the accumulator of tile t - 1, which tile t + 1 takes, has been read
                mbar_arrive(&bars->kv_full[(t + 1) & 1]);
            }
            // uniform across the warp: the TMEM loads below are warp-wide instructions
            // and, as the four warps share the barriers below, a wait that gave up is noted and not repeated
            if (!dead && !__all_sync(0xffffffffu, mbar_wait(&bars->s_full[t & 1], (t >> 1) & 1, p.max_wait))) {
                atomicOr(p.status, kStatusGemmPipeWait);
                dead = true;
            }
            tcgen05_after_sync();
            if (t + 2 < ti.n_tiles) load_keys(t + 2);
            uint32_t s0[32], s1[32];
            tmem_load32(lane + (t & 1) * kBN, s0);
            tmem_load32(lane + (t & 1) * kBN + 32, s1);
            const int key0 = ti.base + t * kBN;
            uint32_t  w[32];
            auto pair = [&](uint32_t x, uint32_t y) {
                const __half2 v = __floats2half2_rn(scaled_sigmoid_log2(fmaf(__uint_as_float(x), scale, bias)),
                                                    scaled_sigmoid_log2(fmaf(__uint_as_float(y), scale, bias)));
                return *reinterpret_cast<const uint32_t*>(&v);
            };
#pragma unroll
            for (int i = 0; i < 16; ++i) w[i] = pair(s0[2 * i], s0[2 * i + 1]), w[16 + i] = pair(s1[2 * i], s1[2 * i + 1]);
            if (!live || key0 < lo || key0 + kBN - 1 > mine) {
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    const int  j  = key0 + 2 * i;
                    const bool in0 = live && j >= lo && j <= mine, in1 = live && j + 1 >= lo && j + 1 <= mine;
                    w[i] = (in0 ? w[i] & 0xffffu : 0u) | (in1 ? w[i] & 0xffff0000u : 0u);
                }
            }
            named_bar_sync(1, kRowThreads);  // the staging buffer has been read
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(out_s + sw_off(tid, c, 0)), "r"(w[4 * c]), "r"(w[4 * c + 1]),
                             "r"(w[4 * c + 2]), "r"(w[4 * c + 3])
                             : "memory");
            }
            named_bar_sync(1, kRowThreads);
#pragma unroll
            for (int r = 0; r < kBM * 8 / kRowThreads; ++r) {
                const int c = tid + r * kRowThreads, row = c >> 3, chunk = c & 7;
                uint4     v;
                asm volatile("ld.shared.v4.b32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "r"(out_s + sw_off(row, chunk, 0)));
                *reinterpret_cast<uint4*>(out + (size_t)row * p.ldk + t * kBN + chunk * 8) = v;
            }
        }
    }
    else if ((tid & 31) == 0) {
        const uint32_t idesc = umma_idesc_bf16(kBM, kBN);
        for (int t = 0; t < ti.n_tiles; ++t) {
            if (!mbar_wait(&bars->kv_full[t & 1], (t >> 1) & 1, p.max_wait)) {
                atomicOr(p.status, kStatusGemmPipeWait);
                break;
            }
            tcgen05_after_sync();
#pragma unroll
            for (int blk = 0; blk < DK / 64; ++blk) {
                const uint64_t dq = umma_desc_k(base + blk * kQBlock), dk = umma_desc_k(k_s + (t & 1) * L::kK + blk * kTBlock);
#pragma unroll
                for (int j = 0; j < 4; ++j) umma_f16_ss(tmem + (t & 1) * kBN, dq + (uint64_t)(2 * j), dk + (uint64_t)(2 * j), idesc, (blk | j) ? 1u : 0u);
            }
            umma_commit(&bars->s_full[t & 1]);
        }
    }
    tcgen05_before_sync();
    __syncthreads();
    if (warp == 4) tmem_free(tmem, 2 * kBN);
}

// ------------------------------------------------------------------------------------------------ mixing across heads
__device__ __forceinline__ void mma_f16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// HB: heads rounded up to 16, in units of 16.  Lane (r = lane / 4, c = lane % 4).  Column n of product t (0..7) is pair
// 8 n + t of the warp's 64, so that a lane's operand halves of all products are 8 consecutive pairs of one head, and a
// lane's results 16 consecutive pairs.
template<int HB>
__global__ void __launch_bounds__(256, HB <= 2 ? 2 : 1) chunk_mix_kernel(const ChunkTcParams p)
{
    pdl_wait();
    pdl_launch_dependents();
    const ChunkAttention& a = p.a;
    const int             warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane >> 2, c = lane & 3, H = a.heads;
    const int             row = blockIdx.x * (8 / kMixSplit) + warp / kMixSplit;
    const TileInfo        ti = tile_info(p, blockIdx.y);
    if (!ti.sp.live || row >= ti.rows) return;
    const int       pos = ti.pos0 + row, seg0 = (chunk_first(pos, a.chunk) - ti.base) / 64, seg1 = (pos - ti.base) / 64;  // beyond: zeros
    const __half*   talk = static_cast<const __half*>(a.talk_half);
    const size_t    head = (size_t)kBM * p.ldk;
    __half*         w    = p.weights + (size_t)blockIdx.y * H * head + (size_t)row * p.ldk;
    uint32_t        tf[HB][HB][4];
#pragma unroll
    for (int m = 0; m < HB; ++m) {
#pragma unroll
        for (int k = 0; k < HB; ++k) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                tf[m][k][e] = *reinterpret_cast<const uint32_t*>(talk + (size_t)(16 * m + r + 8 * (e & 1)) * (16 * HB) + 16 * k + 2 * c + 8 * (e >> 1));
            }
        }
    }
    for (int seg = seg0 + warp % kMixSplit; seg <= seg1; seg += kMixSplit) {
        uint32_t in[HB][4][4];
#pragma unroll
        for (int k = 0; k < HB; ++k) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int   g = 16 * k + 2 * c + (e & 1) + 8 * (e >> 1);
                const uint4 v = g < H ? *reinterpret_cast<const uint4*>(w + g * head + seg * 64 + 8 * r) : make_uint4(0, 0, 0, 0);
                in[k][e][0] = v.x, in[k][e][1] = v.y, in[k][e][2] = v.z, in[k][e][3] = v.w;
            }
        }
        __syncwarp();  // all of the segment is in registers before any of it is written
#pragma unroll
        for (int m = 0; m < HB; ++m) {
            float d[8][4];
#pragma unroll
            for (int t = 0; t < 8; ++t) {
                d[t][0] = d[t][1] = d[t][2] = d[t][3] = 0.f;
                const uint32_t sel = t & 1 ? 0x7632u : 0x5410u;
#pragma unroll
                for (int k = 0; k < HB; ++k) {
                    mma_f16(d[t], tf[m][k], __byte_perm(in[k][0][t >> 1], in[k][1][t >> 1], sel), __byte_perm(in[k][2][t >> 1], in[k][3][t >> 1], sel));
                }
            }
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int h = 16 * m + r + 8 * half;
                uint32_t  o[8];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    o[i]     = pack_bf16(d[2 * i][2 * half], d[2 * i + 1][2 * half]);
                    o[4 + i] = pack_bf16(d[2 * i][2 * half + 1], d[2 * i + 1][2 * half + 1]);
                }
                if (h < H) {
                    asm volatile("st.global.v8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(w + h * head + seg * 64 + 16 * c), "r"(o[0]), "r"(o[1]),
                                 "r"(o[2]), "r"(o[3]), "r"(o[4]), "r"(o[5]), "r"(o[6]), "r"(o[7])
                                 : "memory");
                }
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------ weights times values
struct ValueBars {
    uint64_t full[kStages], done[kStages], o_full;
    uint32_t tmem_base;
};
template<int DV>
struct ValueLayout {
    static constexpr int kP = kBM * kBN * 2, kV = kBN * DV * 2, kStage = kP + kV;
    static constexpr int kSmem = 1024 + kStages * kStage + 128;
};

template<int DV>
__global__ void __launch_bounds__(kThreads, 2) chunk_values_kernel(const ChunkTcParams p)
{
    using L = ValueLayout<DV>;
    using E = __nv_bfloat16;
    extern __shared__ unsigned char smem_dyn[];
    pdl_wait();
    pdl_launch_dependents();
    const ChunkAttention& a = p.a;
    const int             tid = threadIdx.x, warp = tid >> 5, h = blockIdx.x, g = h / (a.heads / a.kv_heads);
    const TileInfo        ti = tile_info(p, blockIdx.y);
    if (!ti.sp.live || ti.rows <= 0) return;
    const uint32_t raw = smem_u32(smem_dyn), base = (raw + 1023u) & ~1023u;
    ValueBars*     bars = reinterpret_cast<ValueBars*>(smem_dyn + (base - raw) + kStages * L::kStage);
    if (tid == 0) {
        for (int i = 0; i < kStages; ++i) mbar_init(&bars->full[i], kRowThreads), mbar_init(&bars->done[i], 1);
        mbar_init(&bars->o_full, 1);
        fence_mbar_init();
    }
    if (warp == 4) tmem_alloc(&bars->tmem_base, DV);
    tcgen05_before_sync();
    __syncthreads();
    tcgen05_after_sync();
    const uint32_t tmem = bars->tmem_base;

    if (warp < 4) {
        const E* vals    = reinterpret_cast<const E*>(ti.sp.slab + a.v_off) + (size_t)g * a.ring * a.vdim;
        const E* weights = reinterpret_cast<const E*>(p.weights) + ((size_t)blockIdx.y * a.heads + h) * kBM * p.ldk;
        bool     ok      = true;
        auto load = [&](int t) {
            if (t < ti.n_tiles) {
                const uint32_t dst  = base + (t % kStages) * L::kStage;
                const int      key0 = ti.base + t * kBN;
                copy_rows<kBM, kBN>(dst, 0, weights + t * kBN, p.ldk, kBM, kBN);
                copy_rows<kBN, DV>(dst + L::kP, kTBlock, vals + (size_t)(key0 % a.ring) * a.vdim, a.vdim, min(kBN, ti.pos1 + 1 - key0), a.vdim);
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        load(0);
        load(1);
        for (int t = 0; t < ti.n_tiles; ++t) {
            // the stage of tile t + 2 was tile t - 1's
            if (t > 0 && t + 2 < ti.n_tiles && !mbar_wait(&bars->done[(t - 1) % kStages], ((t - 1) / kStages) & 1, p.max_wait)) {
                atomicOr(p.status, kStatusGemmPipeWait);
                ok = false;
                break;
            }
            load(t + 2);
            asm volatile("cp.async.wait_group 2;" ::: "memory");
            fence_async_shared();
            mbar_arrive(&bars->full[t % kStages]);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        if (!__all_sync(0xffffffffu, ok && mbar_wait(&bars->o_full, 0, p.max_wait))) atomicOr(p.status, kStatusGemmTmemWait);
        tcgen05_after_sync();
        const bool     live = tid < ti.rows;
        const uint32_t lane = tmem + ((uint32_t)(warp * 32) << 16);
        E*             out  = static_cast<E*>(p.c.out) + (size_t)(ti.sp.tok0 + ti.q0 + tid) * p.c.out_ld;
#pragma unroll 1
        for (int c = 0; c < DV / 32; ++c) {
            uint32_t o[32];
            tmem_load32(lane + 32 * c, o);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                if (!live || 32 * c + 8 * i >= a.vdim) continue;
                auto two = [&](int j) {
                    return pack_bf16(__uint_as_float(o[8 * i + j]) * (1.f / kWeightScale), __uint_as_float(o[8 * i + j + 1]) * (1.f / kWeightScale));
                };
                *reinterpret_cast<uint4*>(out + h * a.vdim + 32 * c + 8 * i) = make_uint4(two(0), two(2), two(4), two(6));
            }
        }
        if (live && h == a.heads - 1) {
            for (int d = a.heads * a.vdim; d < p.c.out_pad; ++d) out[d] = from_f32<E>(0.f);
        }
    }
    else if ((tid & 31) == 0) {
        const uint32_t idesc = umma_idesc_bf16(kBM, DV, true);
        for (int t = 0; t < ti.n_tiles; ++t) {
            if (!mbar_wait(&bars->full[t % kStages], (t / kStages) & 1, p.max_wait)) {
                atomicOr(p.status, kStatusGemmPipeWait);
                break;
            }
            tcgen05_after_sync();
            const uint32_t p_addr = base + (t % kStages) * L::kStage;
            const uint64_t dp = umma_desc_k(p_addr), dv = umma_desc_mn(p_addr + L::kP, kTBlock);
#pragma unroll
            for (int j = 0; j < 4; ++j) umma_f16_ss(tmem, dp + (uint64_t)(2 * j), dv + (uint64_t)(128 * j), idesc, (t | j) ? 1u : 0u);
            umma_commit(&bars->done[t % kStages]);
        }
        umma_commit(&bars->o_full);  // arrives when everything issued so far is complete (also on the give-up path)
    }
    tcgen05_before_sync();
    __syncthreads();
    if (warp == 4) tmem_free(tmem, DV);
}

// keys of a scratch row: a tile's first key is up to 63 before its chunk, its last query up to 127 behind its first
int row_keys(const ChunkAttention& a, int max_context)
{
    const int all = (max_context + kBN - 1) / kBN;
    return kBN * (a.chunk > 0 ? std::min(all, (a.chunk + 189) / kBN + 1) : all);
}
bool sizes_fit(const ChunkAttention& a)
{
    return a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.vdim <= 128 && a.heads <= kMaxHeads;
}

cudaError_t prepare(int)
{
    cudaError_t e = cudaFuncSetAttribute(chunk_scores_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, ScoreLayout<64>::kSmem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(chunk_scores_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, ScoreLayout<128>::kSmem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(chunk_values_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, ValueLayout<64>::kSmem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(chunk_values_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, ValueLayout<128>::kSmem);
    return e;
}
const KernelPreparation g_prepare(prepare);

}  // namespace

size_t chunk_attention_scratch(const ChunkAttention& a, int max_context, bool f32)
{
    return f32 || !sizes_fit(a) ? 0 : (size_t)a.heads * kBM * row_keys(a, max_context) * sizeof(__half);
}

bool chunk_attention_tc_supported(const ChunkAttention& a, const MixerCall& c)
{
    const size_t one = chunk_attention_scratch(a, c.max_context, c.f32);
    return one > 0 && c.tiles && c.tile_count > 0 && a.talk_half && a.weights && a.weights_bytes >= one && a.ring % kBN == 0 && a.q_col % 8 == 0
           && c.proj_ld % 8 == 0 && c.out_ld % 8 == 0;
}

int chunk_attention_tc(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st)
{
    const int     per = (int)std::min<size_t>(65535, a.weights_bytes / chunk_attention_scratch(a, c.max_context, false));
    ChunkTcParams p{a, c, 0, row_keys(a, c.max_context), static_cast<__half*>(a.weights), h->status, kMaxWaitCycles};
    for (; p.tile0 < c.tile_count; p.tile0 += per) {
        const int  items = std::min(per, c.tile_count - p.tile0), hb = talk_pad(a.heads) / 16;
        const dim3 grid(a.heads, items), rows(kBM * kMixSplit / 8, items);
        cudaError_t e = a.dim <= 64 ? launch_kernel(chunk_scores_kernel<64>, grid, dim3(kThreads), ScoreLayout<64>::kSmem, st, c.pdl, p) :
                                      launch_kernel(chunk_scores_kernel<128>, grid, dim3(kThreads), ScoreLayout<128>::kSmem, st, c.pdl, p);
        if (e == cudaSuccess) {
            const auto mix = hb == 1 ? chunk_mix_kernel<1> : hb == 2 ? chunk_mix_kernel<2> : hb == 3 ? chunk_mix_kernel<3> : chunk_mix_kernel<4>;
            e              = launch_kernel(mix, rows, dim3(256), 0, st, c.pdl, p);
        }
        if (e == cudaSuccess) {
            e = a.vdim <= 64 ? launch_kernel(chunk_values_kernel<64>, grid, dim3(kThreads), ValueLayout<64>::kSmem, st, c.pdl, p) :
                               launch_kernel(chunk_values_kernel<128>, grid, dim3(kThreads), ValueLayout<128>::kSmem, st, c.pdl, p);
        }
        if (e != cudaSuccess) {
            h->last_cuda_error = (int)e;
            return TM_ERR_CUDA;
        }
        h->launches += 3;
    }
    return TM_OK;
}

}  // namespace tmb
