// Decode step of the chunk attention (ChunkAttention in mixers.h), bf16: cache append and attention of one new token per
// sequence in one kernel.
//
// CTA = (split of the visible keys, sequence) with all heads, as the weights of all heads meet for every key.  A warp owns
// an item (a kv head x up to 16 of its query heads) and every kw-th block of 16 keys, which it streams through a private
// cp.async ring (16-byte chunks swizzled by row):
//   S[head, key] = Q K^T    mma.m16n8k16, Q fragments in registers, K rows through ldmatrix; sigmoid; fp16 into shared memory
//   P[head, key] = talk W   the weights of all heads for the warp's keys, through ldmatrix.trans
//   O[head, d]  += P V      P straight from the fragments, V rows through ldmatrix.trans
// Weights are not normalised, so warps and splits simply add up: the splits of a cluster through distributed shared memory,
// every CTA a slice of the outputs; clusters of a sequence meet in scratch, slice by slice, and the last CTA to arrive sums
// them in order (no cluster waits for another).  The new token's key and value are read where the projections left them.
// Before griddepcontrol.wait a CTA only reads its span and rows cached by earlier steps.
#include "chunk_attention.h"
#include "common.cuh"
#include "tm_b200.h"

#include <algorithm>

namespace tmb {
namespace {

constexpr int   kKeys = 16, kHeads = 16, kMaxStages = 4, kMaxWarps = 16, kMaxAllHeads = 64, kMaxCluster = 4;
constexpr float kLog2e = 1.4426950408889634f;

struct StepParams {
    ChunkAttention a;
    MixerCall      c;
    int            splits, cluster, head_blocks, items, kw, stages, hb;  // splits: a multiple of cluster
    float*         scratch;  // [sequence][cluster][heads][vdim]
    int*           tickets;  // [sequence][slice]
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
__device__ __forceinline__ float scaled_sigmoid_log2(float x)  // sigmoid of x / log2(e), times kWeightScale
{
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-x));
    return __fdividef(kWeightScale, 1.f + e);
}
__device__ __forceinline__ float load_cluster(uint32_t addr, uint32_t rank)  // shared memory of another CTA of the cluster
{
    float    y;
    uint32_t there;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(there) : "r"(addr), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(y) : "r"(there) : "memory");
    return y;
}
__device__ __forceinline__ void cluster_sync()
{
    asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ void wait_pending(int groups)
{
    switch (groups) {
        case 0: asm volatile("cp.async.wait_group 0;" ::: "memory"); break;
        case 1: asm volatile("cp.async.wait_group 1;" ::: "memory"); break;
        case 2: asm volatile("cp.async.wait_group 2;" ::: "memory"); break;
        default: asm volatile("cp.async.wait_group 3;" ::: "memory"); break;
    }
}
// byte offset of 16-byte chunk `chunk` of row `row`
template<int D>
__device__ __forceinline__ uint32_t sw(int row, int chunk)
{
    return (uint32_t)(row * D * 2 + ((chunk ^ (row & 7)) << 4));
}

template<int D, int MAXT>
__global__ void __launch_bounds__(MAXT) chunk_step_kernel(const StepParams p)
{
    using E             = __nv_bfloat16;
    constexpr int kTile = kKeys * D * 2;  // bytes of a K or V block
    extern __shared__ __align__(128) unsigned char sm[];
    __shared__ int s_last;
    const ChunkAttention& a    = p.a;
    const int             tid = threadIdx.x, threads = blockDim.x, warp = tid >> 5, lane = tid & 31;
    const SeqSpan         sp   = p.c.spans[blockIdx.y];
    const int             item = warp % p.items, kb = warp / p.items;
    const int             g = item / p.head_blocks, group = a.heads / a.kv_heads, in_group = (item % p.head_blocks) * kHeads;
    const int             h0 = g * group + in_group, heads = min(kHeads, group - in_group);
    const int             i = sp.history, first = chunk_first(i, a.chunk);
    const bool            live  = sp.live != 0;
    const int             total = live ? i - first + 1 : 0;  // with the new token, the last
    const int             TK = kKeys * p.kw, tiles = (total + TK - 1) / TK, ST = p.stages;
    const int             b0 = (int)((long long)blockIdx.x * tiles / p.splits), b1 = (int)((long long)(blockIdx.x + 1) * tiles / p.splits);
    const E*              keys = reinterpret_cast<const E*>(sp.slab + a.k_off) + (size_t)g * a.ring * a.dim;
    const E*              vals = reinterpret_cast<const E*>(sp.slab + a.v_off) + (size_t)g * a.ring * a.vdim;
    const E*              row  = static_cast<const E*>(p.c.proj) + (size_t)sp.tok0 * p.c.proj_ld;
    const int             slot0 = first % a.ring;  // the visible tokens span less than a ring
    const int             w_ld  = TK + 8;          // halves
    __half* const         wbuf  = reinterpret_cast<__half*>(sm);  // [2][16 hb][w_ld]
    const uint32_t        wbytes = (uint32_t)(2 * 16 * p.hb * w_ld * 2), sm_b = smem_u32(sm), ring_off = (wbytes + 127u) & ~127u;
    const uint32_t        ring = sm_b + ring_off + (uint32_t)warp * ST * 2 * kTile;

    auto fetch = [&](int b, int stage) {
        const uint32_t dst = ring + stage * 2 * kTile;
        if (b < b1) {
#pragma unroll
            for (int r = 0; r < kKeys * D / 8 / 32; ++r) {
                const int  c = lane + r * 32, rw = c / (D / 8), chunk = c % (D / 8), idx = b * TK + kb * kKeys + rw;
                const bool in = idx < total, fresh = idx == total - 1 && a.writes;
                int        slot = slot0 + idx;
                if (slot >= a.ring) slot -= a.ring;
                const bool ok_k = in && chunk * 8 < a.dim, ok_v = in && chunk * 8 < a.vdim;
                const E*   k = fresh ? row + a.k_col + g * a.dim : keys + (in ? (size_t)slot * a.dim : 0);
                const E*   v = fresh ? row + a.v_col + g * a.vdim : vals + (in ? (size_t)slot * a.vdim : 0);
                cp_async16z(dst + sw<D>(rw, chunk), k + (ok_k ? chunk * 8 : 0), ok_k ? 16 : 0);
                cp_async16z(dst + kTile + sw<D>(rw, chunk), v + (ok_v ? chunk * 8 : 0), ok_v ? 16 : 0);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // rows of earlier steps: no kernel of this step writes what is read here
    int ahead = 0;
    for (; ahead < ST && (b0 + ahead + 1) * TK < total; ++ahead) fetch(b0 + ahead, ahead);
    for (int w = tid; w < (int)wbytes / 4; w += threads) reinterpret_cast<uint32_t*>(sm)[w] = 0u;
    uint32_t tf[kMaxAllHeads / 16][4];  // rows of the mixing matrix that belong to the item's heads
    const int r = lane >> 2, c2 = 2 * (lane & 3);
#pragma unroll
    for (int k = 0; k < kMaxAllHeads / 16; ++k) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int hh = r + 8 * (e & 1);
            tf[k][e]     = k < p.hb && hh < heads ?
                               *reinterpret_cast<const uint32_t*>(static_cast<const __half*>(a.talk_half) + (size_t)(h0 + hh) * 16 * p.hb + 16 * k + c2 + 8 * (e >> 1)) :
                               0u;
        }
    }
    float bias[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) bias[e] = r + 8 * e < heads ? a.bias[h0 + r + 8 * e] * kLog2e : 0.f;
    const float scale = a.scale * kLog2e;
    pdl_wait();
    pdl_launch_dependents();
    if (!live) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        return;
    }
    for (; ahead < ST; ++ahead) fetch(b0 + ahead, ahead);
    uint32_t q[D / 16][4];
#pragma unroll
    for (int k = 0; k < D / 16; ++k) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int hh = r + 8 * (e & 1), d = 16 * k + c2 + 8 * (e >> 1);
            q[k][e]      = hh < heads && d < a.dim ? *reinterpret_cast<const uint32_t*>(row + a.q_col + (h0 + hh) * a.dim + d) : 0u;
        }
    }
    __syncthreads();  // wbuf is zero
    float o[D / 8][4];
#pragma unroll
    for (int n = 0; n < D / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    int stage = 0;
    for (int b = b0; b < b1; ++b) {
        wait_pending(ST - 1);
        __syncwarp();
        const uint32_t kt = ring + stage * 2 * kTile, vt = kt + kTile;
        float          s[2][4] = {};
#pragma unroll
        for (int k = 0; k < D / 16; ++k) {
            uint32_t f[4];  // keys 0-7 / d low, keys 0-7 / d high, keys 8-15 / d low, keys 8-15 / d high
            ldsm4(kt + sw<D>((lane & 7) + ((lane >> 4) << 3), 2 * k + ((lane >> 3) & 1)), f);
            mma_bf16(s[0], q[k], f[0], f[1]);
            mma_bf16(s[1], q[k], f[2], f[3]);
        }
        __half* const w = wbuf + (b & 1) * 16 * p.hb * w_ld;
#pragma unroll
        for (int t = 0; t < 2; ++t) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                if (r + 8 * e >= heads) continue;
                const int   idx = b * TK + kb * kKeys + 8 * t + c2;
                const float x = idx < total ? scaled_sigmoid_log2(fmaf(s[t][2 * e], scale, bias[e])) : 0.f;
                const float y = idx + 1 < total ? scaled_sigmoid_log2(fmaf(s[t][2 * e + 1], scale, bias[e])) : 0.f;
                *reinterpret_cast<__half2*>(w + (h0 + r + 8 * e) * w_ld + kb * kKeys + 8 * t + c2) = __floats2half2_rn(x, y);
            }
        }
        __syncthreads();  // one per tile: the buffer of tile b is written again at tile b + 2, behind the barrier of tile b + 1
        float m[2][4] = {};
#pragma unroll
        for (int k = 0; k < kMaxAllHeads / 16; ++k) {
            if (k >= p.hb) break;
            uint32_t f[4];  // heads 0-7 / keys 0-7, heads 8-15 / keys 0-7, the same for keys 8-15
            ldsm4t(smem_u32(w + (16 * k + (lane & 15)) * w_ld + kb * kKeys + 8 * (lane >> 4)), f);
            mma_m16n8k16(m[0], tf[k], f[0], f[1]);
            mma_m16n8k16(m[1], tf[k], f[2], f[3]);
        }
        const uint32_t pf[4] = {pack_bf16(m[0][0], m[0][1]), pack_bf16(m[0][2], m[0][3]), pack_bf16(m[1][0], m[1][1]), pack_bf16(m[1][2], m[1][3])};
#pragma unroll
        for (int n = 0; n < D / 8; n += 2) {
            uint32_t f[4];  // keys 0-7 / d low, keys 8-15 / d low, keys 0-7 / d high, keys 8-15 / d high
            ldsm4t(vt + sw<D>(lane & 15, n + (lane >> 4)), f);
            mma_bf16(o[n], pf, f[0], f[1]);
            mma_bf16(o[n + 1], pf, f[2], f[3]);
        }
        __syncwarp();
        fetch(b + ST, stage);
        stage = stage + 1 == ST ? 0 : stage + 1;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // the rings are free: they take the warps' results

    float* const all = reinterpret_cast<float*>(sm + ring_off);  // [warp][16][D]
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        float* rec = all + ((size_t)warp * kHeads + r + 8 * e) * D;
#pragma unroll
        for (int n = 0; n < D / 8; ++n) *reinterpret_cast<float2*>(rec + 8 * n + c2) = make_float2(o[n][2 * e], o[n][2 * e + 1]);
    }
    const int  rank = (int)blockIdx.x % p.cluster, n = a.heads * a.vdim, x0 = rank * n / p.cluster, x1 = (rank + 1) * n / p.cluster;
    E* const   out  = static_cast<E*>(p.c.out) + (size_t)sp.tok0 * p.c.out_ld;
    const bool whole = p.splits == p.cluster;  // one cluster has all of the sequence
    if (p.cluster > 1) {
        cluster_sync();
    }
    else {
        __syncthreads();
    }
    float* const recs = p.scratch + (size_t)blockIdx.y * (p.splits / p.cluster) * n;
    for (int x = x0 + tid; x < x1; x += threads) {
        const int h = x / a.vdim, in = h % group, it = h / group * p.head_blocks + in / kHeads;
        float     y = 0.f;
        if (p.cluster > 1) {
            float v[kMaxCluster];
            for (int k = 0; k < p.kw; ++k) {
                const uint32_t at = smem_u32(all + ((size_t)(k * p.items + it) * kHeads + in % kHeads) * D + x % a.vdim);
#pragma unroll
                for (int c = 0; c < kMaxCluster; ++c) v[c] = c < p.cluster ? load_cluster(at, c) : 0.f;
#pragma unroll
                for (int c = 0; c < kMaxCluster; ++c) y += v[c];
            }
        }
        else {
            for (int k = 0; k < p.kw; ++k) y += all[((size_t)(k * p.items + it) * kHeads + in % kHeads) * D + x % a.vdim];
        }
        y *= 1.f / kWeightScale;
        if (whole) {
            out[x] = from_f32<E>(y);
        }
        else {
            __stcg(recs + (blockIdx.x / p.cluster) * n + x, y);
        }
    }
    if (!whole) {
        const int clusters = p.splits / p.cluster;
        __threadfence();
        __syncthreads();
        if (tid == 0) {
            int* ticket = p.tickets + blockIdx.y * p.cluster + rank;
            s_last      = atomicAdd(ticket, 1) == clusters - 1;
            if (s_last) *ticket = 0;
        }
        __syncthreads();
        if (s_last) {
            __threadfence();
            for (int x = x0 + tid; x < x1; x += threads) {
                float y = 0.f;
#pragma unroll 8
                for (int k = 0; k < clusters; ++k) y += __ldcg(recs + (size_t)k * n + x);
                out[x] = from_f32<E>(y);
            }
        }
    }
    // ---- off the critical path: cache append, padding columns
    if ((int)blockIdx.x == p.splits - 1) {
        if (a.writes) {
            const int slot = i % a.ring;
            E *       kw   = reinterpret_cast<E*>(sp.slab + a.k_off), *vw = reinterpret_cast<E*>(sp.slab + a.v_off);
            for (int x = tid; x < a.kv_heads * a.dim; x += threads) kw[((size_t)(x / a.dim) * a.ring + slot) * a.dim + x % a.dim] = row[a.k_col + x];
            for (int x = tid; x < a.kv_heads * a.vdim; x += threads) vw[((size_t)(x / a.vdim) * a.ring + slot) * a.vdim + x % a.vdim] = row[a.v_col + x];
        }
        for (int d = a.heads * a.vdim + tid; d < p.c.out_pad; d += threads) out[d] = from_f32<E>(0.f);
    }
    if (p.cluster > 1) cluster_sync();  // the others have read this CTA's results
}

struct StepPlan {
    int D = 0, head_blocks = 0, items = 0, kw = 0, stages = 0, hb = 0;
    size_t smem = 0;
};
StepPlan plan_of(const tm_handle* h, const ChunkAttention& a)
{
    StepPlan p;
    p.D           = a.dim <= 64 && a.vdim <= 64 ? 64 : 128;
    p.head_blocks = (a.heads / a.kv_heads + kHeads - 1) / kHeads;
    p.items       = a.kv_heads * p.head_blocks;
    p.hb          = talk_pad(a.heads) / 16;
    p.kw          = std::max(1, 8 / p.items);
    const int    warps = p.items * p.kw;
    const size_t fixed = ((size_t)2 * 16 * p.hb * (kKeys * p.kw + 8) * 2 + 127) / 128 * 128, stage = (size_t)warps * 2 * kKeys * p.D * 2;
    if (warps > kMaxWarps || fixed + stage + 256 > (size_t)h->max_smem) return p;
    p.stages = (int)std::min<size_t>(kMaxStages, (h->max_smem - 256 - fixed) / stage);
    p.smem   = fixed + p.stages * stage;
    return p;
}

template<int D, int MAXT>
cudaError_t launch(const StepParams& p, int batch, size_t smem, cudaStream_t st)
{
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(p.splits, batch), cfg.blockDim = dim3(p.items * p.kw * 32), cfg.dynamicSmemBytes = smem, cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id                                         = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x                           = p.cluster;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id                                         = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs                                          = attr;
    cfg.numAttrs                                       = p.c.pdl ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, chunk_step_kernel<D, MAXT>, p);
}

cudaError_t prepare(int max_smem)
{
    cudaError_t e = cudaSuccess;
    for (const void* f : {(const void*)chunk_step_kernel<64, 256>, (const void*)chunk_step_kernel<128, 256>, (const void*)chunk_step_kernel<64, 512>,
                          (const void*)chunk_step_kernel<128, 512>}) {
        if (e == cudaSuccess) e = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem - 256);
    }
    return e;
}
const KernelPreparation g_prepare(prepare);

}  // namespace

bool chunk_attention_step_supported(const tm_handle* h, const ChunkAttention& a, const MixerCall& c)
{
    return !c.f32 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.vdim <= 128 && a.heads <= kMaxAllHeads && a.talk_half && a.q_col % 8 == 0
           && (!a.writes || (a.k_col % 8 == 0 && a.v_col % 8 == 0)) && c.proj_ld % 8 == 0 && plan_of(h, a).stages > 0;
}

int chunk_attention_step(tm_handle* h, const ChunkAttention& a, const MixerCall& c, cudaStream_t st)
{
    const StepPlan  pl = plan_of(h, a);
    StepParams      p{a, c, 1, 1, pl.head_blocks, pl.items, pl.kw, pl.stages, pl.hb, static_cast<float*>(h->attn_scratch), h->attn_counters};
    // one wave of CTAs, a split with at least two tiles; the bound on the visible keys is the host's
    const long long keys = a.chunk > 0 ? std::min(a.chunk, c.max_context) : c.max_context, resident = std::max<long long>(1, h->max_smem / (long long)pl.smem);
    const long long splits = std::min(std::min(resident, 2ll) * h->sm_count / c.batch, keys / (2 * kKeys * pl.kw));
    while (p.cluster < kMaxCluster && 2 * p.cluster <= splits) p.cluster *= 2;
    long long clusters = std::max<long long>(1, splits / p.cluster);
    clusters = std::min<long long>(clusters, (long long)(h->attn_scratch_bytes / ((size_t)c.batch * a.heads * a.vdim * 4)));
    if (clusters < 1 || (long long)c.batch * p.cluster > (long long)h->attn_counter_ints) clusters = 1;
    p.splits = (int)clusters * p.cluster;
    const bool        wide = pl.items * pl.kw > 8;
    const cudaError_t e = pl.D == 64 ? (wide ? launch<64, 512>(p, c.batch, pl.smem, st) : launch<64, 256>(p, c.batch, pl.smem, st)) :
                                       (wide ? launch<128, 512>(p, c.batch, pl.smem, st) : launch<128, 256>(p, c.batch, pl.smem, st));
    if (e != cudaSuccess) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    ++h->launches;
    return TM_OK;
}

}  // namespace tmb
