// Config-driven decoder (decoder.h): set-up, weights, prefill passes and the decode step.
#include "decoder.h"
#include "common.cuh"
#include "numeric.cuh"
#include "safetensors.h"
#include "step_kernels.h"

#include <algorithm>
#include <cmath>
#include <cstring>

using namespace tmb;

namespace tmb {
namespace {

constexpr int kDefaultPrefill = 4096;
constexpr int kWantRows       = 256;  // rows of one lm-head product of a prefill

int round_up(int x, int m)
{
    return (x + m - 1) / m * m;
}
size_t round_up_bytes(size_t x)
{
    return (x + 255) / 256 * 256;
}

// x row (from the embedding when ids are given), its copy in the element type and its sum of squares: one CTA per token
template<typename E>
__global__ void __launch_bounds__(256) rows_kernel(float* x, E* xb, float* ssq, const E* embed, const int* ids, float scale, int width, int x_ld,
                                                   int vocab)
{
    __shared__ float red[8];
    pdl_wait();
    pdl_launch_dependents();
    const int t  = blockIdx.x;
    float*    xr = x + (size_t)t * width;
    E*        br = xb + (size_t)t * x_ld;
    const E*  er = ids ? embed + (size_t)min(max(ids[t], 0), vocab - 1) * width : nullptr;
    float     sq = 0.f;
    if (width % 4 == 0 && x_ld % 4 == 0) {
        for (int i = 4 * threadIdx.x; i < width; i += 1024) {
            float4 v;
            if (er) {
                v = make_float4(to_f32(er[i]) * scale, to_f32(er[i + 1]) * scale, to_f32(er[i + 2]) * scale, to_f32(er[i + 3]) * scale);
                *reinterpret_cast<float4*>(xr + i) = v;
            }
            else {
                v = *reinterpret_cast<const float4*>(xr + i);
            }
            if constexpr (sizeof(E) == 2) {
                *reinterpret_cast<uint2*>(br + i) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
            }
            else {
                *reinterpret_cast<float4*>(br + i) = v;
            }
            sq += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        }
    }
    else {
        for (int i = threadIdx.x; i < width; i += 256) {
            const float v = er ? to_f32(er[i]) * scale : xr[i];
            if (er) xr[i] = v;
            br[i] = from_f32<E>(v);
            sq += v * v;
        }
    }
    sq = warp_sum(sq);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
    __syncthreads();
    if (threadIdx.x == 0) {
        float s = 0.f;
        for (int i = 0; i < 8; ++i) s += red[i];
        ssq[t] = s;
    }
}

// rows `want[i]` of xb / ssq -> row i of the gathered copies
template<typename E>
__global__ void gather_rows_kernel(E* dst, float* dst_ssq, const E* xb, const float* ssq, const int* want, int x_ld)
{
    const int i = blockIdx.x, t = want[i];
    for (int c = threadIdx.x; c < x_ld; c += blockDim.x) dst[(size_t)i * x_ld + c] = xb[(size_t)t * x_ld + c];
    if (threadIdx.x == 0) dst_ssq[i] = ssq[t];
}

// one span and one input token per sequence of a decode step
__global__ void step_spans_kernel(const tm_llama_decode_state st, const int* picked, int* ids, unsigned char* inactive, SeqSpan* spans, int vocab,
                                  int session_len)
{
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b >= st.batch_size) return;
    bool      off = false;
    const int id  = step_input(st.step, st.start_step, st.forced_ids, picked, b, st.batch_size, st.max_steps, vocab, &off);
    const int len = st.sequence_lengths[b];
    ids[b]        = id;
    inactive[b]   = off ? 1 : 0;
    SeqSpan s;
    s.slab    = static_cast<unsigned char*>(st.k_cache_ptrs[b]);
    s.history = len;
    s.n       = 1;
    s.tok0    = b;
    s.live    = !off && len < session_len ? 1 : 0;
    spans[b]  = s;
}

__device__ __forceinline__ float hash_normal(unsigned long long seed, unsigned long long i)
{
    auto mix = [](unsigned long long z) {  // splitmix64 finaliser
        z = (z ^ (z >> 30)) * 0xbf58476d1ce4e5b9ull;
        z = (z ^ (z >> 27)) * 0x94d049bb133111ebull;
        return z ^ (z >> 31);
    };
    const unsigned long long r = mix(seed + 0x9e3779b97f4a7c15ull * (i + 1));
    const float u = ((unsigned)(r >> 40) + 1) * (1.f / 16777217.f), v = (unsigned)((r >> 8) & 0xffffff) * (1.f / 16777216.f);
    return sqrtf(-2.f * logf(u)) * cospif(2.f * v);
}
template<typename E>
__global__ void random_kernel(E* dst, long long rows, long long cols, long long row_stride, float mean, float std, unsigned long long seed)
{
    const long long n = rows * cols;
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        dst[(i / cols) * row_stride + i % cols] = from_f32<E>(mean + std * hash_normal(seed, (unsigned long long)i));
    }
}

// talk [heads][heads] -> fp16 [pad][pad], zeros beyond
__global__ void talk_half_kernel(__half* dst, const float* talk, int heads, int pad)
{
    for (int i = threadIdx.x; i < pad * pad; i += blockDim.x) {
        const int h = i / pad, g = i % pad;
        dst[i] = __float2half_rn(h < heads && g < heads ? talk[h * heads + g] : 0.f);
    }
}

float half_to_float(uint16_t h)
{
    const int   e = (h >> 10) & 31, m = h & 1023;
    const float v = e == 0 ? std::ldexp((float)m, -24) : (e == 31 ? (m ? NAN : INFINITY) : std::ldexp((float)(m + 1024), e - 25));
    return h & 0x8000 ? -v : v;
}
float element_as_float(const unsigned char* p, const std::string& dtype)
{
    if (dtype == "F32") {
        float f;
        std::memcpy(&f, p, 4);
        return f;
    }
    uint16_t h;
    std::memcpy(&h, p, 2);
    if (dtype == "F16") return half_to_float(h);
    const uint32_t w = (uint32_t)h << 16;
    float          f;
    std::memcpy(&f, &w, 4);
    return f;
}
uint16_t float_to_bf16(float f)
{
    uint32_t w;
    std::memcpy(&w, &f, 4);
    if ((w & 0x7fffffffu) > 0x7f800000u) return 0x7fff;
    return (uint16_t)((w + 0x7fffu + ((w >> 16) & 1)) >> 16);
}

}  // namespace
}  // namespace tmb

bool tm_decoder::alloc(void** p, size_t bytes)
{
    bytes = std::max<size_t>(bytes, 256);
    if (cudaMalloc(p, bytes) != cudaSuccess) {
        *p = nullptr;
        cudaGetLastError();
        return false;
    }
    owned.push_back(*p);
    return cudaMemset(*p, 0, bytes) == cudaSuccess;
}

tm_decoder::~tm_decoder()
{
    graph.drop();
    for (void* p : owned) cudaFree(p);
}

int tm_decoder::init(tm_handle* handle, const DecoderConfig& c, const tm_model_options& opt)
{
    h              = handle;
    cfg            = c;
    f32            = opt.dtype == TM_DTYPE_F32;
    vocab_size     = c.vocab;
    max_batch_size = opt.max_batch_size;
    session_len    = opt.session_len;
    max_prefill    = std::min(opt.max_prefill_tokens > 0 ? opt.max_prefill_tokens : kDefaultPrefill, std::max(16, session_len * max_batch_size));
    int prev = 0;
    cudaGetDevice(&prev);
    cudaSetDevice(h->device);
    const size_t es = f32 ? 4 : 2;
    const int    W = c.width, tokens = std::max(max_prefill, max_batch_size);
    bool         ok = true;
    x_ld            = round_up(W, 8);
    size_t off      = 0;
    size_t delta_floats = 0;  // of a prefill, per token
    auto   take = [&](size_t bytes) {
        const size_t at = off;
        off             = round_up_bytes(off + bytes);
        return at;
    };
    auto target = [&](const std::string& name, int64_t rows, int64_t cols, void* dst, int64_t stride) -> WeightTarget& {
        WeightTarget t;
        t.name = name, t.rows = rows, t.cols = cols, t.dst = dst, t.row_stride = stride;
        t.init_std = 1.f / std::sqrt((float)cols);
        targets.push_back(t);
        return targets.back();
    };
    auto vec = [&](const std::string& name, int64_t n, float** dst, float mean, float std) {
        ok             = ok && alloc((void**)dst, n * 4);
        WeightTarget& t = target(name, 1, n, *dst, n);
        t.vector = true, t.f32 = true, t.init_mean = mean, t.init_std = std;
    };
    auto gain = [&](const std::string& name, float** dst) {
        vec(name, 1, dst, 1.f, 0.f);
        targets.back().scalar = true;
    };
    auto at = [&](void* base, int64_t row, int64_t ld, int64_t col = 0) { return static_cast<char*>(base) + (size_t)(row * ld + col) * es; };

    const bool gated = c.form == LayerForm::kGatedBranches;
    // longest chunk of any layer that reads a layer's keys: the ring has to keep it
    std::vector<int> reach(c.layers.size(), 0);
    for (size_t i = 0; i < c.layers.size(); ++i) {
        const MixerSpec& m = c.layers[i].mixer;
        int&             r = reach[m.kv_from >= 0 ? (size_t)m.kv_from : i];
        r                  = std::max(r, m.chunk > 0 ? m.chunk : session_len);
    }
    int top_max = 0, ff_max = 0, experts_max = 0, router_max = 0;
    layers.resize(c.layers.size());
    for (size_t i = 0; i < layers.size() && ok; ++i) {
        DecoderLayer&     L = layers[i];
        const MixerSpec&  m = c.layers[i].mixer;
        const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
        L.spec              = c.layers[i];
        const int ff        = L.spec.ff;
        int       cols      = 0;
        auto      segment   = [&](int n) {
            const int at0 = cols;
            cols += round_up(n, 8);
            return at0;
        };
        struct Part {
            const char* name;
            int         rows, col;
        };
        std::vector<Part> parts;
        if (m.type == MixerType::kAttention) {
            WindowAttention& a = L.attention;
            a.heads = m.heads, a.kv_heads = m.kv_heads, a.dim = m.dim, a.vdim = m.vdim, a.rot_dims = m.rot_dims;
            a.scale = (float)m.scale, a.softcap = (float)m.softcap, a.window = m.window, a.pool = m.pool;
            a.q_col = segment(m.heads * m.dim), a.k_col = segment(m.kv_heads * m.dim), a.v_col = segment(m.kv_heads * m.vdim);
            a.g_col = segment(m.heads);
            parts   = {{"q", m.heads * m.dim, a.q_col}, {"k", m.kv_heads * m.dim, a.k_col}, {"v", m.kv_heads * m.vdim, a.v_col}, {"g", m.heads, a.g_col}};
            // the oldest query of a pass still sees its window, and the pass completes blocks that began before it
            const long long keep = (long long)std::max(m.window, m.pool) + max_prefill;
            a.ring               = round_up((int)std::min<long long>(m.window > 0 ? keep : session_len, session_len), 128);
            a.pool_rows          = m.pool > 0 ? round_up(std::max(1, session_len / m.pool), 8) : 0;
            a.k_off              = take((size_t)m.kv_heads * a.ring * m.dim * es);
            a.v_off              = take((size_t)m.kv_heads * a.ring * m.vdim * es);
            a.pk_off             = take((size_t)m.kv_heads * a.pool_rows * m.dim * es);
            a.pv_off             = take((size_t)m.kv_heads * a.pool_rows * m.vdim * es);
            std::vector<float> f(std::max(1, m.rot_dims / 2));
            for (int k = 0; k < m.rot_dims / 2; ++k) f[k] = (float)(std::pow(m.rot_base, -2.0 * k / m.rot_dims) / m.rot_factor);
            ok = ok && alloc((void**)&L.inv_freq, f.size() * 4) && cudaMemcpy(L.inv_freq, f.data(), f.size() * 4, cudaMemcpyHostToDevice) == cudaSuccess;
            a.inv_freq = L.inv_freq;
        }
        else if (m.type == MixerType::kGeneralDelta) {
            DeltaRule& d = L.delta;
            const int  n = m.heads * m.dim;
            d.heads = m.heads, d.dim = m.dim, d.rank = m.rank, d.norm_eps = (float)c.norm_eps;
            d.r_col = segment(n), d.k_col = segment(n), d.v_col = segment(n), d.a_col = segment(n), d.g_col = segment(n), d.w1_col = segment(m.rank);
            parts = {{"r", n, d.r_col}, {"k", n, d.k_col}, {"v", n, d.v_col}, {"a", n, d.a_col}, {"g", n, d.g_col}, {"w1", m.rank, d.w1_col}};
            L.tanh_lo = d.w1_col, L.tanh_hi = d.w1_col + m.rank;
            d.w2_ld     = round_up(m.rank, 8);
            d.state_off = take((size_t)m.heads * m.dim * m.dim * 4);
            ok          = ok && alloc(&L.w2, (size_t)n * d.w2_ld * es);
            target(mp + "w2", n, m.rank, L.w2, d.w2_ld);
            vec(mp + "w0", n, &L.w0, 0.f, 1.f);
            vec(mp + "a.b", n, &L.a_bias, 0.f, 1.f);
            vec(mp + "norm", n, &L.norm, 1.f, 0.f);
            d.w2 = L.w2, d.w0 = L.w0, d.a_bias = L.a_bias, d.norm = L.norm;
            delta_floats = std::max(delta_floats, delta_rule_scratch_floats(d));
        }
        else if (m.type == MixerType::kChunkAttention) {
            ChunkAttention& a = L.chunk;
            a.heads = m.heads, a.kv_heads = m.kv_heads, a.dim = m.dim, a.vdim = m.vdim, a.scale = (float)m.scale, a.chunk = m.chunk;
            a.writes = m.kv_from < 0;
            a.q_col  = segment(m.heads * m.dim);
            parts    = {{"q", m.heads * m.dim, a.q_col}};
            if (a.writes) {
                a.k_col = segment(m.kv_heads * m.dim), a.v_col = segment(m.kv_heads * m.vdim);
                parts.push_back({"k", m.kv_heads * m.dim, a.k_col});
                parts.push_back({"v", m.kv_heads * m.vdim, a.v_col});
                a.ring  = round_up((int)std::min<long long>((long long)reach[i] + max_prefill, session_len), 128);
                a.k_off = take((size_t)m.kv_heads * a.ring * m.dim * es);
                a.v_off = take((size_t)m.kv_heads * a.ring * m.vdim * es);
            }
            else {
                const ChunkAttention& o = layers[m.kv_from].chunk;
                a.ring = o.ring, a.k_off = o.k_off, a.v_off = o.v_off;
            }
            const int pad = talk_pad(m.heads);
            ok = ok && alloc((void**)&L.talk, (size_t)m.heads * m.heads * 4) && alloc(&L.talk_half, (size_t)pad * pad * 2);
            vec(mp + "pb", m.heads, &L.bias, -3.f, 1.f);
            target(mp + "talk", m.heads, m.heads, L.talk, m.heads).f32 = true;
            a.bias = L.bias, a.talk = L.talk, a.talk_half = L.talk_half;
            attention_weights_bytes = std::max(attention_weights_bytes, chunk_attention_scratch(a, session_len, f32));
        }
        else {
            GatedLinear& d = L.linear;
            const int    n = m.heads * m.dim, nv = m.heads * m.vdim;
            d.heads = m.heads, d.dim = m.dim, d.vdim = m.vdim, d.rank = m.rank, d.norm_eps = (float)c.norm_eps, d.tau = (float)m.tau;
            d.scale = (float)(1.0 / std::sqrt((double)m.dim));
            d.q_col = segment(n), d.k_col = segment(n), d.v_col = segment(nv), d.g_col = segment(nv), d.a_col = segment(m.rank);
            parts   = {{"q", n, d.q_col}, {"k", n, d.k_col}, {"v", nv, d.v_col}, {"g", nv, d.g_col}, {"a1", m.rank, d.a_col}};
            d.w2_ld     = round_up(m.rank, 8);
            d.state_off = take((size_t)m.heads * m.dim * m.vdim * 4);
            ok          = ok && alloc(&L.w2, (size_t)n * d.w2_ld * es);
            target(mp + "a2", n, m.rank, L.w2, d.w2_ld);
            vec(mp + "a2.b", n, &L.a_bias, 2.f, 1.f);
            vec(mp + "norm", m.vdim, &L.norm, 1.f, 0.f);
            d.w2 = L.w2, d.bias = L.a_bias, d.norm = L.norm;
            delta_floats = std::max(delta_floats, gated_linear_scratch_floats(d));
        }
        if (gated) {
            const MoeSpec& e = L.spec.moe;
            L.rg1_col        = segment(W);
            L.in_rows        = round_up(cols, kDenseTile);
            if (e.experts > 0) {
                L.x2_from = cols = L.in_rows;
                L.rg2_col = segment(W), L.router_col = segment(e.experts + e.identity);
                L.in_rows = cols;
            }
            L.mix_pad = round_up(m.out_width(), 8);
            L.out_k   = L.mix_pad;
            ok = ok && alloc(&L.w_in, (size_t)L.in_rows * x_ld * es) && alloc(&L.w_out, (size_t)W * L.out_k * es);
            if (!ok) break;
            vec(p + "norm1", W, &L.norm1, 1.f, 0.1f);
            for (const Part& q : parts) target(mp + q.name, q.rows, W, at(L.w_in, q.col, x_ld), x_ld);
            target(mp + "o", W, m.out_width(), L.w_out, L.out_k);
            target(p + "rg1", W, W, at(L.w_in, L.rg1_col, x_ld), x_ld);
            vec(p + "rg1.b", W, &L.rg1_bias, 0.f, 1.f);
            if (e.experts > 0) {
                const int n = e.experts + e.identity, down_ld = round_up(e.ff, 8);
                L.router = {e.experts, e.identity, e.top, e.groups, e.keep, nullptr};
                ok = ok && alloc(&L.w_experts, (size_t)e.experts * 2 * e.ff * x_ld * es) && alloc(&L.w_down, (size_t)e.experts * W * down_ld * es);
                if (!ok) break;
                vec(p + "norm2", W, &L.norm2, 1.f, 0.1f);
                target(p + "rg2", W, W, at(L.w_in, L.rg2_col, x_ld), x_ld);
                vec(p + "rg2.b", W, &L.rg2_bias, 0.f, 1.f);
                target(p + "mlp.router", n, W, at(L.w_in, L.router_col, x_ld), x_ld);
                vec(p + "mlp.correction", n, &L.correction, 0.f, 0.f);
                L.router.correction = L.correction;
                for (int x = 0; x < e.experts; ++x) {
                    const std::string ep = p + "mlp.e" + std::to_string(x) + ".";
                    target(ep + "gate", e.ff, W, at(L.w_experts, (int64_t)x * 2 * e.ff, x_ld), 2 * x_ld);
                    target(ep + "up", e.ff, W, at(L.w_experts, (int64_t)x * 2 * e.ff + 1, x_ld), 2 * x_ld);
                    target(ep + "down", W, e.ff, at(L.w_down, (int64_t)x * W, down_ld), down_ld);
                }
                top_max = std::max(top_max, e.top), ff_max = std::max(ff_max, e.ff), experts_max = std::max(experts_max, e.experts);
                router_max = std::max(router_max, n);
            }
            proj_ld = std::max(proj_ld, round_up(L.x2_from > 0 ? L.router_col : L.in_rows, 8));
            y_ld    = std::max(y_ld, L.out_k);
            continue;
        }
        L.mixer_cols = round_up(cols, kDenseTile);
        L.in_rows    = L.mixer_cols + 2 * ff;
        L.mix_pad    = round_up(m.out_width(), 8);
        L.out_k      = L.mix_pad + ff;
        ok = ok && alloc(&L.w_in, (size_t)L.in_rows * x_ld * es) && alloc(&L.w_out, (size_t)W * round_up(L.out_k, 8) * es);
        if (!ok) break;
        gain(p + "norm1", &L.gain);
        for (const Part& q : parts) target(mp + q.name, q.rows, W, at(L.w_in, q.col, x_ld), x_ld);
        target(mp + "o", W, m.out_width(), L.w_out, round_up(L.out_k, 8)).init_std *= 0.5f;
        if (ff > 0) {
            target(p + "mlp.gate", ff, W, at(L.w_in, L.mixer_cols, x_ld), 2 * x_ld);
            target(p + "mlp.up", ff, W, at(L.w_in, L.mixer_cols + 1, x_ld), 2 * x_ld);
            target(p + "mlp.down", W, ff, at(L.w_out, 0, 0, L.mix_pad), round_up(L.out_k, 8)).init_std *= 0.5f;
        }
        proj_ld = std::max(proj_ld, L.mixer_cols);
        y_ld    = std::max(y_ld, round_up(L.out_k, 8));
    }
    slab = std::max<size_t>(off, 256);
    ok   = ok && alloc(&embed, (size_t)c.vocab * W * es) && alloc(&head, (size_t)c.vocab * x_ld * es);
    if (ok) {
        target("embed", c.vocab, W, embed, W).init_std = 1.f;
        target("head", c.vocab, W, head, x_ld);
        if (gated) {
            vec("final.norm", W, &final_norm, 1.f, 0.1f);
        }
        else {
            gain("final.norm", &final_gain);
        }
    }
    ssq_stride            = round_up(tokens, 8);
    const size_t T        = (size_t)tokens, column_tiles = (size_t)(W + kDenseTile - 1) / kDenseTile;
    const size_t logit_rows = (size_t)max_batch_size;
    ok = ok && alloc((void**)&x, T * W * 4) && alloc((void**)&ssq, column_tiles * ssq_stride * 4) && alloc(&xb, T * x_ld * es)
         && alloc(&proj, T * proj_ld * es) && alloc(&y, T * y_ld * es) && alloc((void**)&delta_scratch, (size_t)max_prefill * delta_floats * 4) && alloc((void**)&logits, logit_rows * c.vocab * 4)
         && alloc(&want_xb, (size_t)kWantRows * x_ld * es) && alloc((void**)&want_ssq, (size_t)kWantRows * 4) && alloc((void**)&ids, T * 4)
         && alloc((void**)&want, T * 4) && alloc((void**)&picked, T * 4) && alloc((void**)&inactive, T) && alloc((void**)&spans, T * sizeof(SeqSpan));
    if (gated) {
        const size_t rows = T * std::max(1, top_max);
        router_ld = round_up(std::max(1, router_max), 4), act_ld = round_up(std::max(1, ff_max), 8);
        moe_rows.ld = x_ld;
        // as many query tiles at a time as a pass has, within 1 GB
        const size_t most = T / 128 + max_batch_size;
        if (attention_weights_bytes > 0) attention_weights_bytes *= std::max<size_t>(1, std::min(most, ((size_t)1 << 30) / attention_weights_bytes));
        ok = ok && alloc(&xb2, T * x_ld * es) && alloc((void**)&tiles, T * sizeof(QueryTile));
        if (top_max > 0) {
            ok = ok && alloc(&expert_act, rows * act_ld * es) && alloc(&expert_out, rows * W * es) && alloc((void**)&router_logits, T * router_ld * 4)
                 && alloc((void**)&moe_rows.counts, (size_t)experts_max * 4) && alloc((void**)&moe_rows.offsets, (size_t)(experts_max + 1) * 4)
                 && alloc((void**)&moe_rows.slots, rows * 4) && alloc((void**)&moe_rows.weights, rows * 4) && alloc((void**)&moe_rows.ranks, rows * 4)
                 && alloc(&moe_rows.sorted, rows * x_ld * es);
        }
        if (attention_weights_bytes > 0) ok = ok && alloc(&attention_weights, attention_weights_bytes);
        for (DecoderLayer& L : layers) L.chunk.weights = attention_weights, L.chunk.weights_bytes = attention_weights_bytes;
    }
    const cudaError_t e = cudaGetLastError();
    cudaSetDevice(prev);
    if (!ok) {
        h->last_cuda_error = (int)e;
        return TM_ERR_CUDA;
    }
    return TM_OK;
}

int tm_decoder::load(const std::string& path, std::string* why)
{
    SafeTensors st;
    if (!st.open(path)) {
        *why = "cannot read " + path;
        return TM_ERR_IO;
    }
    int prev = 0;
    cudaGetDevice(&prev);
    cudaSetDevice(h->device);
    int                        rc = TM_OK;
    std::vector<unsigned char> raw, converted;
    for (const WeightTarget& t : targets) {
        const SafeTensor* s     = st.find(t.name);
        bool              match = s && (s->dtype == "BF16" || s->dtype == "F32" || s->dtype == "F16");
        if (match) {
            if (t.scalar) {
                match = s->count() == 1;
            }
            else if (t.vector) {
                match = s->shape.size() == 1 && s->shape[0] == t.cols;
            }
            else {
                match = s->shape.size() == 2 && s->shape[0] == t.rows && s->shape[1] == t.cols;
            }
        }
        if (!match || !st.read(*s, raw)) {
            *why = (s ? "tensor of another shape or type: " : "missing tensor: ") + t.name;
            rc   = TM_ERR_IO;
            break;
        }
        const size_t n = (size_t)(t.rows * t.cols), in = s->dtype == "F32" ? 4 : 2, es = t.f32 || f32 ? 4 : 2;
        const void*  src = raw.data();
        if (!(es == 4 && s->dtype == "F32") && !(es == 2 && s->dtype == "BF16")) {
            converted.resize(n * es);
            for (size_t i = 0; i < n; ++i) {
                const float v = element_as_float(raw.data() + i * in, s->dtype);
                if (es == 4) {
                    std::memcpy(converted.data() + i * 4, &v, 4);
                }
                else {
                    const uint16_t b = float_to_bf16(v);
                    std::memcpy(converted.data() + i * 2, &b, 2);
                }
            }
            src = converted.data();
        }
        if (cudaMemcpy2D(t.dst, (size_t)t.row_stride * es, src, (size_t)t.cols * es, (size_t)t.cols * es, (size_t)t.rows, cudaMemcpyHostToDevice)
            != cudaSuccess) {
            *why = "copy to the device failed: " + t.name;
            rc   = TM_ERR_CUDA;
            break;
        }
    }
    if (rc == TM_OK) rc = derive_weights();
    cudaSetDevice(prev);
    return rc;
}

// what kernels want in another form than the checkpoint has it
int tm_decoder::derive_weights()
{
    for (const DecoderLayer& L : layers) {
        if (L.talk_half) talk_half_kernel<<<1, 256>>>(static_cast<__half*>(L.talk_half), L.talk, L.chunk.heads, talk_pad(L.chunk.heads));
    }
    return cudaDeviceSynchronize() == cudaSuccess ? TM_OK : TM_ERR_CUDA;
}

int tm_decoder::random_weights(unsigned long long seed)
{
    int prev = 0;
    cudaGetDevice(&prev);
    cudaSetDevice(h->device);
    unsigned long long k = seed * 1000003ull;
    for (const WeightTarget& t : targets) {
        k += 7919;
        if (t.f32 || f32) {
            random_kernel<float><<<1024, 256>>>(static_cast<float*>(t.dst), t.rows, t.cols, t.row_stride, t.init_mean, t.init_std, k);
        }
        else {
            random_kernel<__nv_bfloat16><<<1024, 256>>>(static_cast<__nv_bfloat16*>(t.dst), t.rows, t.cols, t.row_stride, t.init_mean, t.init_std, k);
        }
    }
    const int rc = derive_weights();
    cudaSetDevice(prev);
    return rc;
}

int tm_decoder::new_cache(tm_cache_manager** out, size_t max_entry_count, size_t chunk_size) const
{
    return tm_cache_manager_create_slabs(out, slab, (size_t)session_len, max_entry_count, chunk_size, h->device);
}

// The tokens of one pass through the layers; spans, ids are on the device already
struct tm_decoder::Pass {
    int  batch = 0, tokens = 0, max_n = 0;
    bool decode = false, fold = false, pdl = false;
    bool need_output = true;        // whether anybody reads what the last layer leaves
    // after every layer: residual rows out (prefill, optional)
    float* const* residual_rows = nullptr;  // [batch] destination of each span's rows of layer 0
    size_t        residual_layer_stride = 0;
    const SeqSpan* host_spans = nullptr;
    int            tile_count = 0;          // prefill: query tiles on the device
};

int tm_decoder::run_mixer(const DecoderLayer& L, const Pass& p, cudaStream_t s)
{
    MixerCall c;
    c.proj = proj, c.proj_ld = proj_ld, c.out = y, c.out_ld = y_ld, c.out_pad = L.mix_pad, c.spans = spans, c.batch = p.batch;
    c.tokens = p.tokens, c.max_n = p.max_n, c.max_context = session_len, c.f32 = f32, c.pdl = p.pdl;
    if (tiles && !p.decode) c.tiles = tiles, c.tile_count = p.tile_count;
    switch (L.spec.mixer.type) {
        case MixerType::kAttention: return p.decode ? window_attention_decode(h, L.attention, c, s) : window_attention_prefill(h, L.attention, c, s);
        case MixerType::kGeneralDelta: return p.decode ? delta_rule_decode(h, L.delta, c, s) : delta_rule_prefill(h, L.delta, c, delta_scratch, s);
        case MixerType::kChunkAttention: return p.decode ? chunk_attention_decode(h, L.chunk, c, s) : chunk_attention_prefill(h, L.chunk, c, s);
        default: return p.decode ? gated_linear_decode(h, L.linear, c, s) : gated_linear_prefill(h, L.linear, c, delta_scratch, s);
    }
}

int tm_decoder::copy_residual(const Pass& p, size_t layer, cudaStream_t s)
{
    for (int b = 0; p.residual_rows && b < p.batch; ++b) {
        if (cudaMemcpyAsync(p.residual_rows[b] + layer * p.residual_layer_stride, x + (size_t)p.host_spans[b].tok0 * cfg.width,
                            (size_t)p.host_spans[b].n * cfg.width * 4, cudaMemcpyDeviceToDevice, s)
            != cudaSuccess) {
            return TM_ERR_CUDA;
        }
    }
    return TM_OK;
}

// LayerForm::kGatedBranches; leaves the final norm's rows in xb
int tm_decoder::run_gated_layers(const Pass& p, cudaStream_t s)
{
    const int    W   = cfg.width;
    const size_t es  = f32 ? 4 : 2;
    const bool   pdl = p.pdl;
    const float  mult = (float)cfg.residual_mult;
    // the rows kernel ahead of layer `next` (the output behind the last), with what the layer before leaves to add
    auto rows = [&](size_t next) {
        RowsCall c;
        c.x = x, c.tokens = p.tokens, c.width = W, c.eps = (float)cfg.norm_eps, c.out_a = xb, c.out_ld = x_ld;
        if (next == 0) {
            c.embed = embed, c.ids = ids, c.vocab = cfg.vocab;
        }
        else if (layers[next - 1].router.experts > 0) {
            const DecoderLayer& L = layers[next - 1];
            c.expert_rows = expert_out, c.input = xb2, c.input_ld = x_ld, c.slots = moe_rows.slots, c.weights = moe_rows.weights, c.top = L.router.top;
            c.gate = static_cast<char*>(proj) + (size_t)L.rg2_col * es, c.gate_ld = proj_ld, c.gate_bias = L.rg2_bias, c.mult = mult;
        }
        c.weight_a = next < layers.size() ? layers[next].norm1 : final_norm;
        if (next < layers.size() && layers[next].router.experts > 0) c.weight_b = layers[next].norm2, c.out_b = xb2;
        c.clear = moe_rows.counts;
        for (const DecoderLayer& L : layers) c.clear_count = std::max(c.clear_count, L.router.experts);
        return norm_rows(h, c, f32, s, pdl);
    };
    int rc = rows(0);
    for (size_t l = 0; l < layers.size() && rc == TM_OK; ++l) {
        const DecoderLayer& L = layers[l];
        DenseGemm           g;
        g.w = L.w_in, g.ldw = x_ld, g.x = xb, g.ldx = x_ld, g.tokens = p.tokens, g.n_out = L.in_rows, g.k = W;
        g.ep.kind = DenseKind::kStore, g.ep.out = proj, g.ep.out_ld = proj_ld;
        if (L.x2_from > 0) {
            g.x2 = xb2, g.x2_from = L.x2_from;
            g.ep.f32_out = router_logits, g.ep.f32_from = L.router_col, g.ep.f32_ld = router_ld;
            g.n_out = L.router_col + L.router.outputs();
        }
        if ((rc = dense_gemm(h, g, f32, s, pdl)) != TM_OK) break;
        rc = run_mixer(L, p, s);
        if (rc != TM_OK || (l + 1 == layers.size() && !p.need_output)) break;

        DenseGemm o;
        o.w = L.w_out, o.ldw = L.out_k, o.x = y, o.ldx = y_ld, o.tokens = p.tokens, o.n_out = W, o.k = L.out_k;
        o.ep.kind = DenseKind::kResidual, o.ep.residual = x, o.ep.residual_ld = W, o.ep.mult = mult;
        o.ep.gate = static_cast<char*>(proj) + (size_t)L.rg1_col * es, o.ep.gate_ld = proj_ld, o.ep.gate_bias = L.rg1_bias;
        if ((rc = dense_gemm(h, o, f32, s, pdl)) != TM_OK) break;
        if (L.router.experts > 0) {
            const MoeSpec& e = L.spec.moe;
            if ((rc = moe_dispatch(h, L.router, moe_rows, router_logits, router_ld, xb2, p.tokens, W, f32, s, pdl)) != TM_OK) break;
            DenseGemm u;
            u.w = L.w_experts, u.ldw = x_ld, u.x = moe_rows.sorted, u.ldx = x_ld, u.tokens = p.tokens * e.top, u.n_out = 2 * e.ff, u.k = W;
            u.groups.count = e.experts, u.groups.offsets = moe_rows.offsets;
            u.ep.kind = DenseKind::kInput, u.ep.split = 0, u.ep.act = expert_act, u.ep.act_ld = act_ld;
            u.ep.activation = DenseActivation::kClampedSwish, u.ep.limit = (float)e.limit, u.ep.slope = kSwishSlope;
            if ((rc = dense_gemm(h, u, f32, s, pdl)) != TM_OK) break;
            DenseGemm d;
            d.w = L.w_down, d.ldw = round_up(e.ff, 8), d.x = expert_act, d.ldx = act_ld, d.tokens = u.tokens, d.n_out = W, d.k = e.ff;
            d.groups = u.groups;
            d.ep.kind = DenseKind::kStore, d.ep.out = expert_out, d.ep.out_ld = W;
            if ((rc = dense_gemm(h, d, f32, s, pdl)) != TM_OK) break;
        }
        if ((rc = rows(l + 1)) != TM_OK) break;
        rc = copy_residual(p, l, s);
    }
    return rc;
}

int tm_decoder::run_layers(const Pass& p, cudaStream_t s)
{
    if (cfg.form == LayerForm::kGatedBranches) return run_gated_layers(p, s);
    const int  W   = cfg.width;
    const bool pdl = p.pdl;
    auto rows = [&](const int* token_ids) {
        cudaError_t e;
        if (f32) {
            e = launch_kernel(rows_kernel<float>, dim3(p.tokens), dim3(256), 0, s, pdl, x, static_cast<float*>(xb), ssq, static_cast<const float*>(embed),
                              token_ids, (float)cfg.embedding_scale, W, x_ld, cfg.vocab);
        }
        else {
            using B = __nv_bfloat16;
            e = launch_kernel(rows_kernel<B>, dim3(p.tokens), dim3(256), 0, s, pdl, x, static_cast<B*>(xb), ssq, static_cast<const B*>(embed), token_ids,
                              (float)cfg.embedding_scale, W, x_ld, cfg.vocab);
        }
        ++h->launches;
        return e == cudaSuccess ? TM_OK : TM_ERR_CUDA;
    };
    int rc = rows(ids);
    int ssq_parts = 1;
    for (size_t l = 0; l < layers.size() && rc == TM_OK; ++l) {
        const DecoderLayer& L    = layers[l];
        const bool          last = l + 1 == layers.size();
        DenseGemm           g;
        g.w = L.w_in, g.ldw = x_ld, g.x = xb, g.ldx = x_ld, g.tokens = p.tokens, g.n_out = L.in_rows, g.k = W;
        g.ep.kind = DenseKind::kInput;
        g.ep.ssq = ssq, g.ep.ssq_parts = ssq_parts, g.ep.ssq_stride = ssq_stride, g.ep.inv_width = 1.f / (float)W, g.ep.eps = (float)cfg.norm_eps;
        g.ep.gain = L.gain;
        g.ep.out = proj, g.ep.out_ld = proj_ld, g.ep.tanh_lo = L.tanh_lo, g.ep.tanh_hi = L.tanh_hi, g.ep.split = L.mixer_cols;
        g.ep.act = static_cast<char*>(y) + (size_t)L.mix_pad * (f32 ? 4 : 2), g.ep.act_ld = y_ld;
        if ((rc = dense_gemm(h, g, f32, s, pdl)) != TM_OK) break;

        rc = run_mixer(L, p, s);
        if (rc != TM_OK || (last && !p.need_output)) break;

        DenseGemm o;
        o.w = L.w_out, o.ldw = round_up(L.out_k, 8), o.x = y, o.ldx = y_ld, o.tokens = p.tokens, o.n_out = W, o.k = L.out_k;
        o.ep.kind = DenseKind::kResidual, o.ep.residual = x, o.ep.residual_ld = W;
        if (p.fold) {
            o.ep.cast = xb, o.ep.cast_ld = x_ld, o.ep.ssq_out = ssq, o.ep.ssq_out_stride = ssq_stride;
            ssq_parts = (W + kDenseTile - 1) / kDenseTile;
        }
        if ((rc = dense_gemm(h, o, f32, s, pdl)) != TM_OK) break;
        if ((rc = copy_residual(p, l, s)) != TM_OK) break;
        if (!p.fold) rc = rows(nullptr);
    }
    return rc;
}

int tm_decoder::prefill(const tm_model_prefill_state& st, cudaStream_t s)
{
    const int B = st.batch_size, total = st.cu_seqlens[B];
    if (total == 0) return TM_OK;
    const size_t V = (size_t)cfg.vocab, W = (size_t)cfg.width;
    std::vector<int> done(B, 0);
    for (int left = total; left > 0;) {
        // ---- one pass: the sequences in turn, each with as many of its tokens as still fit
        std::vector<SeqSpan> sp;
        std::vector<int>     tok, wanted, want_seq_begin;  // wanted: rows of this pass
        std::vector<float*>  res_rows, logit_rows;         // destination per span
        Pass                 p;
        for (int b = 0; b < B && p.tokens < max_prefill; ++b) {
            const int begin = st.cu_seqlens[b] + done[b], n = std::min(st.cu_seqlens[b + 1] - begin, max_prefill - p.tokens);
            if (n <= 0) continue;
            SeqSpan q;
            q.slab = static_cast<unsigned char*>(st.k_cache[b]), q.history = st.history_lengths[b] + done[b], q.n = n, q.tok0 = p.tokens, q.live = 1;
            tok.insert(tok.end(), st.input_ids + begin, st.input_ids + begin + n);
            want_seq_begin.push_back((int)wanted.size());
            const int* lo = std::lower_bound(st.want, st.want + st.want_count, begin);
            const int* hi = std::lower_bound(st.want, st.want + st.want_count, begin + n);
            logit_rows.push_back(st.logits_out + (size_t)(lo - st.want) * V);
            for (; lo < hi; ++lo) wanted.push_back(*lo - begin + p.tokens);
            if (st.residual_out) res_rows.push_back(st.residual_out + (size_t)begin * W);
            sp.push_back(q);
            p.tokens += n;
            p.max_n = std::max(p.max_n, n);
            done[b] += n;
        }
        want_seq_begin.push_back((int)wanted.size());
        left -= p.tokens;
        p.batch       = (int)sp.size();
        p.need_output = !wanted.empty() || st.residual_out != nullptr;
        p.host_spans  = sp.data();
        std::vector<QueryTile> query_tiles;
        for (int b = 0; tiles && b < p.batch; ++b) {
            for (int q = 0; q < sp[b].n; q += 128) query_tiles.push_back({b, q});
        }
        p.tile_count = (int)query_tiles.size();
        if (st.residual_out) p.residual_rows = res_rows.data(), p.residual_layer_stride = (size_t)total * W;
        if (cudaMemcpyAsync(spans, sp.data(), sp.size() * sizeof(SeqSpan), cudaMemcpyHostToDevice, s) != cudaSuccess
            || cudaMemcpyAsync(ids, tok.data(), tok.size() * 4, cudaMemcpyHostToDevice, s) != cudaSuccess
            || (tiles && cudaMemcpyAsync(tiles, query_tiles.data(), query_tiles.size() * sizeof(QueryTile), cudaMemcpyHostToDevice, s) != cudaSuccess)
            || (!wanted.empty() && cudaMemcpyAsync(want, wanted.data(), wanted.size() * 4, cudaMemcpyHostToDevice, s) != cudaSuccess)) {
            return TM_ERR_CUDA;
        }
        int rc = run_layers(p, s);
        // ---- logits of the wanted rows: per span, so that they land where the caller's order puts them
        for (int b = 0; b < p.batch && rc == TM_OK; ++b) {
            for (int w = want_seq_begin[b]; w < want_seq_begin[b + 1] && rc == TM_OK; w += kWantRows) {
                const int n = std::min(kWantRows, want_seq_begin[b + 1] - w);
                if (f32) {
                    gather_rows_kernel<float><<<n, 128, 0, s>>>(static_cast<float*>(want_xb), want_ssq, static_cast<const float*>(xb), ssq, want + w, x_ld);
                }
                else {
                    using E = __nv_bfloat16;
                    gather_rows_kernel<E><<<n, 128, 0, s>>>(static_cast<E*>(want_xb), want_ssq, static_cast<const E*>(xb), ssq, want + w, x_ld);
                }
                ++h->launches;
                DenseGemm g;
                g.w = head, g.ldw = x_ld, g.x = want_xb, g.ldx = x_ld, g.tokens = n, g.n_out = cfg.vocab, g.k = cfg.width;
                g.ep.kind = DenseKind::kF32, g.ep.out = logit_rows[b] + (size_t)(w - want_seq_begin[b]) * V, g.ep.out_ld = cfg.vocab;
                if (cfg.form == LayerForm::kScalarNorm) {
                    g.ep.ssq = want_ssq, g.ep.ssq_parts = 1, g.ep.ssq_stride = kWantRows, g.ep.inv_width = 1.f / (float)W, g.ep.eps = (float)cfg.norm_eps;
                    g.ep.gain = final_gain;
                }
                rc        = dense_gemm(h, g, f32, s, false);
            }
        }
        if (rc != TM_OK) return rc;
    }
    return TM_OK;
}

int tm_decoder::step(const tm_llama_decode_state& st, cudaStream_t s, unsigned long long* launches)
{
    const unsigned long long before = h->launches;
    const int                B      = st.batch_size;
    step_spans_kernel<<<(B + 127) / 128, 128, 0, s>>>(st, picked, ids, inactive, spans, cfg.vocab, session_len);
    if (cudaPeekAtLastError() != cudaSuccess) return TM_ERR_CUDA;
    Pass p;
    p.batch = B, p.tokens = B, p.max_n = 1, p.decode = true, p.fold = !f32 && h->fold_norm, p.pdl = h->pdl != 0;
    int rc = run_layers(p, s);
    if (rc != TM_OK) return rc;
    float*    out = st.logits_out ? st.logits_out : logits;
    DenseGemm g;
    g.w = head, g.ldw = x_ld, g.x = xb, g.ldx = x_ld, g.tokens = B, g.n_out = cfg.vocab, g.k = cfg.width;
    g.ep.kind = DenseKind::kF32, g.ep.out = out, g.ep.out_ld = cfg.vocab;
    if (cfg.form == LayerForm::kScalarNorm) {
        g.ep.ssq = ssq, g.ep.ssq_parts = p.fold ? (cfg.width + kDenseTile - 1) / kDenseTile : 1, g.ep.ssq_stride = ssq_stride;
        g.ep.inv_width = 1.f / (float)cfg.width, g.ep.eps = (float)cfg.norm_eps, g.ep.gain = final_gain;
    }
    if ((rc = dense_gemm(h, g, f32, s, p.pdl)) != TM_OK) return rc;
    if (step_argmax(out, picked, st.output_ids, st.step, inactive, B, cfg.vocab, 1, st.max_steps, s) != cudaSuccess
        || step_advance(st.step, st.sequence_lengths, inactive, B, s) != cudaSuccess) {
        return TM_ERR_CUDA;
    }
    *launches = h->launches - before + 3;
    return TM_OK;
}

int tm_decoder::decode(const tm_llama_decode_state& st, int n_steps, bool use_graph, cudaStream_t s)
{
    if (st.hidden_out) return TM_ERR_UNSUPPORTED;
    return graph.run(h, st, n_steps, use_graph, s, &launches_of_last, [&](unsigned long long* n) { return step(st, s, n); });
}

// ---------------------------------------------------------------------------------------------------- mechanisms alone
namespace {

// `bytes` of the handle's operator buffer, on 256-byte boundaries
bool operator_buffer(tm_handle* h, size_t bytes)
{
    if (bytes <= h->op_buffer_bytes) return true;
    if (h->op_buffer) cudaFree(h->op_buffer);  // waits for the work that uses it
    h->op_buffer = nullptr, h->op_buffer_bytes = 0;
    if (cudaMalloc(&h->op_buffer, bytes) != cudaSuccess) return false;
    h->op_buffer_bytes = bytes;
    return true;
}

// Spans and query tiles of a call on the device, and scratch behind them, in the handle's operator buffer
struct DeviceSpans {
    MixerCall c;
    void*     scratch = nullptr;
    int       rc      = TM_OK;

    // scratch_bytes(call) -> bytes, asked when the call's sizes are known
    template<typename Bytes>
    DeviceSpans(tm_handle* h, const tm_mixer_call& call, cudaStream_t s, Bytes scratch_bytes)
    {
        if (!call.proj || !call.out || call.batch <= 0 || !call.history || !call.n || !call.slabs
            || (call.dtype != TM_DTYPE_BF16 && call.dtype != TM_DTYPE_F32)) {
            rc = TM_ERR_INVALID_ARG;
            return;
        }
        std::vector<SeqSpan> sp(call.batch);
        for (int b = 0; b < call.batch; ++b) {
            if (!call.slabs[b] || call.history[b] < 0 || call.n[b] < 0 || (call.decode && call.n[b] != 1)) rc = TM_ERR_INVALID_ARG;
            sp[b].slab = static_cast<unsigned char*>(call.slabs[b]), sp[b].history = call.history[b], sp[b].n = call.n[b];
            sp[b].tok0 = c.tokens, sp[b].live = 1;
            c.tokens += call.n[b];
            c.max_n       = std::max(c.max_n, call.n[b]);
            c.max_context = std::max(c.max_context, call.history[b] + call.n[b]);
        }
        if (rc == TM_OK && c.tokens == 0) rc = TM_ERR_INVALID_ARG;
        if (rc != TM_OK) return;
        std::vector<QueryTile> tiles;
        for (int b = 0; !call.decode && b < call.batch; ++b) {
            for (int q = 0; q < call.n[b]; q += 128) tiles.push_back({b, q});
        }
        c.proj = call.proj, c.proj_ld = call.proj_ld, c.out = call.out, c.out_ld = call.out_ld, c.batch = call.batch;
        c.f32 = call.dtype == TM_DTYPE_F32, c.tile_count = (int)tiles.size();
        const size_t spans_bytes = round_up_bytes(sp.size() * sizeof(SeqSpan)), tiles_bytes = round_up_bytes(tiles.size() * sizeof(QueryTile));
        if (!operator_buffer(h, spans_bytes + tiles_bytes + scratch_bytes(c))) {
            rc = TM_ERR_CUDA;
            return;
        }
        SeqSpan* d = static_cast<SeqSpan*>(h->op_buffer);
        void* const t = static_cast<char*>(h->op_buffer) + spans_bytes;
        scratch       = static_cast<char*>(t) + tiles_bytes;
        c.spans = d, c.tiles = static_cast<QueryTile*>(t);
        if (cudaMemcpyAsync(d, sp.data(), sp.size() * sizeof(SeqSpan), cudaMemcpyHostToDevice, s) != cudaSuccess
            || (!tiles.empty() && cudaMemcpyAsync(t, tiles.data(), tiles.size() * sizeof(QueryTile), cudaMemcpyHostToDevice, s) != cudaSuccess)) {
            rc = TM_ERR_CUDA;
        }
    }
};

}  // namespace

extern "C" int tm_window_attention(tm_handle* h, const tm_window_attention_params* q, const tm_mixer_call* call, void* stream)
{
    if (!h || !q || !call) return TM_ERR_INVALID_ARG;
    const cudaStream_t s = (cudaStream_t)stream;
    DeviceSpans        sp(h, *call, s, [](const MixerCall&) { return (size_t)0; });
    if (sp.rc != TM_OK) return sp.rc;
    WindowAttention a;
    a.heads = q->heads, a.kv_heads = q->kv_heads, a.dim = q->dim, a.vdim = q->vdim, a.rot_dims = q->rot_dims, a.inv_freq = q->inv_freq;
    a.scale = q->scale, a.softcap = q->softcap, a.window = q->window, a.pool = q->pool, a.ring = q->ring, a.pool_rows = q->pool_rows;
    a.k_off = q->k_off, a.v_off = q->v_off, a.pk_off = q->pooled_k_off, a.pv_off = q->pooled_v_off;
    a.q_col = q->q_col, a.k_col = q->k_col, a.v_col = q->v_col, a.g_col = q->g_col;
    for (int b = 0; b < call->batch; ++b) {
        // everything a query of the call may see has to be in the ring and in the pooled rows
        const int end = call->history[b] + call->n[b], need = a.window > 0 ? std::min(end, std::max(a.window, a.pool) + call->n[b]) : end;
        if (need > a.ring || (a.pool > 0 && end / a.pool > a.pool_rows)) return TM_ERR_INVALID_ARG;
    }
    return call->decode ? window_attention_decode(h, a, sp.c, s) : window_attention_prefill(h, a, sp.c, s);
}

extern "C" int tm_delta_rule(tm_handle* h, const tm_delta_rule_params* q, const tm_mixer_call* call, void* stream)
{
    if (!h || !q || !call || !q->w2 || !q->w0 || !q->a_bias || !q->norm) return TM_ERR_INVALID_ARG;
    const cudaStream_t s = (cudaStream_t)stream;
    DeltaRule          d;
    d.heads = q->heads, d.dim = q->dim, d.rank = q->rank, d.w2 = q->w2, d.w2_ld = q->w2_ld, d.w0 = q->w0, d.a_bias = q->a_bias, d.norm = q->norm;
    d.norm_eps = q->norm_eps, d.unit_eps = q->unit_eps, d.decay_scale = q->decay_scale, d.state_off = q->state_off;
    d.r_col = q->r_col, d.k_col = q->k_col, d.v_col = q->v_col, d.a_col = q->a_col, d.g_col = q->g_col, d.w1_col = q->w1_col;
    DeviceSpans sp(h, *call, s, [&](const MixerCall& c) { return call->decode ? 0 : delta_rule_scratch_floats(d) * sizeof(float) * c.tokens; });
    if (sp.rc != TM_OK) return sp.rc;
    return call->decode ? delta_rule_decode(h, d, sp.c, s) : delta_rule_prefill(h, d, sp.c, static_cast<float*>(sp.scratch), s);
}

extern "C" int tm_chunk_attention(tm_handle* h, const tm_chunk_attention_params* q, const tm_mixer_call* call, void* stream)
{
    if (!h || !q || !call || !q->bias || !q->talk || q->heads <= 0 || q->heads > 1024) return TM_ERR_INVALID_ARG;
    const cudaStream_t s = (cudaStream_t)stream;
    ChunkAttention     a;
    a.heads = q->heads, a.kv_heads = q->kv_heads, a.dim = q->dim, a.vdim = q->vdim, a.scale = q->scale, a.chunk = q->chunk, a.bias = q->bias;
    a.talk = q->talk, a.writes = !q->reads_only, a.ring = q->ring, a.k_off = q->k_off, a.v_off = q->v_off;
    a.q_col = q->q_col, a.k_col = q->k_col, a.v_col = q->v_col;
    const int    pad        = talk_pad(a.heads);
    const size_t talk_bytes = round_up_bytes((size_t)pad * pad * 2);
    DeviceSpans  sp(h, *call, s, [&](const MixerCall& c) {
        a.weights_bytes = call->decode ? 0 : chunk_attention_scratch(a, c.max_context, c.f32) * (q->query_tiles > 0 ? std::min(q->query_tiles, c.tile_count) : c.tile_count);
        return talk_bytes + a.weights_bytes;
    });
    if (sp.rc != TM_OK) return sp.rc;
    for (int b = 0; b < call->batch; ++b) {
        // everything a query of the call may see has to be in the ring
        const int end = call->history[b] + call->n[b], need = a.chunk > 0 ? std::min(end, a.chunk - 1 + call->n[b]) : end;
        if (need > a.ring) return TM_ERR_INVALID_ARG;
    }
    a.talk_half = q->talk_half;
    if (!a.talk_half) {
        a.talk_half = sp.scratch;
        talk_half_kernel<<<1, 256, 0, s>>>(static_cast<__half*>(sp.scratch), a.talk, a.heads, pad);
    }
    a.weights = static_cast<char*>(sp.scratch) + talk_bytes;
    return call->decode ? chunk_attention_decode(h, a, sp.c, s) : chunk_attention_prefill(h, a, sp.c, s);
}

extern "C" int tm_gated_linear(tm_handle* h, const tm_gated_linear_params* q, const tm_mixer_call* call, void* stream)
{
    if (!h || !q || !call || !q->w2 || !q->bias || !q->norm || !(q->tau > 0.f)) return TM_ERR_INVALID_ARG;
    const cudaStream_t s = (cudaStream_t)stream;
    GatedLinear        d;
    d.heads = q->heads, d.dim = q->dim, d.vdim = q->vdim, d.rank = q->rank, d.w2 = q->w2, d.w2_ld = q->w2_ld, d.bias = q->bias, d.norm = q->norm;
    d.norm_eps = q->norm_eps, d.scale = q->scale, d.tau = q->tau, d.state_off = q->state_off;
    d.q_col = q->q_col, d.k_col = q->k_col, d.v_col = q->v_col, d.g_col = q->g_col, d.a_col = q->a_col;
    DeviceSpans sp(h, *call, s, [&](const MixerCall& c) { return call->decode ? 0 : gated_linear_scratch_floats(d) * sizeof(float) * c.tokens; });
    if (sp.rc != TM_OK) return sp.rc;
    return call->decode ? gated_linear_decode(h, d, sp.c, s) : gated_linear_prefill(h, d, sp.c, static_cast<float*>(sp.scratch), s);
}

extern "C" int tm_moe(tm_handle* h, const tm_moe_params* q, void* stream)
{
    if (!h || !q || !q->x || !q->logits || !q->input || !q->gate || !q->gate_bias || !q->correction || !q->w_experts || !q->w_down || q->tokens < 0
        || q->experts <= 0 || q->top <= 0 || (q->dtype != TM_DTYPE_BF16 && q->dtype != TM_DTYPE_F32)) {
        return TM_ERR_INVALID_ARG;
    }
    if (q->tokens == 0) return TM_OK;
    const cudaStream_t s   = (cudaStream_t)stream;
    const bool         f32 = q->dtype == TM_DTYPE_F32;
    const size_t       es = f32 ? 4 : 2, T = (size_t)q->tokens, rows = T * q->top;
    const int          act_ld = round_up(q->ff, 8);
    size_t             at     = 0;
    auto take = [&](size_t bytes) {
        const size_t begin = at;
        at += round_up_bytes(bytes);
        return begin;
    };
    const size_t counts = take((size_t)q->experts * 4), offsets = take((size_t)(q->experts + 1) * 4), slots = take(rows * 4), weights = take(rows * 4),
                 ranks = take(rows * 4), sorted = take(rows * q->input_ld * es), act = take(rows * act_ld * es), out = take(rows * q->width * es);
    if (!operator_buffer(h, at)) return TM_ERR_CUDA;
    char* const base = static_cast<char*>(h->op_buffer);
    MoeRows     m;
    m.counts = (int*)(base + counts), m.offsets = (int*)(base + offsets), m.slots = (int*)(base + slots), m.weights = (float*)(base + weights);
    m.ranks = (int*)(base + ranks), m.sorted = base + sorted, m.ld = q->input_ld;
    const MoeRouter r{q->experts, q->identity, q->top, q->groups, q->keep, q->correction};
    if (cudaMemsetAsync(m.counts, 0, (size_t)q->experts * 4, s) != cudaSuccess) return TM_ERR_CUDA;
    int rc = moe_dispatch(h, r, m, q->logits, q->logits_ld, q->input, q->tokens, q->width, f32, s, false);
    if (rc != TM_OK) return rc;
    DenseGemm u;
    u.w = q->w_experts, u.ldw = q->input_ld, u.x = m.sorted, u.ldx = m.ld, u.tokens = (int)rows, u.n_out = 2 * q->ff, u.k = q->width;
    u.groups.count = q->experts, u.groups.offsets = m.offsets;
    u.ep.kind = DenseKind::kInput, u.ep.act = base + act, u.ep.act_ld = act_ld;
    u.ep.activation = DenseActivation::kClampedSwish, u.ep.limit = q->limit, u.ep.slope = q->slope;
    if ((rc = dense_gemm(h, u, f32, s, false)) != TM_OK) return rc;
    DenseGemm d;
    d.w = q->w_down, d.ldw = act_ld, d.x = base + act, d.ldx = act_ld, d.tokens = (int)rows, d.n_out = q->width, d.k = q->ff, d.groups = u.groups;
    d.ep.kind = DenseKind::kStore, d.ep.out = base + out, d.ep.out_ld = q->width;
    if ((rc = dense_gemm(h, d, f32, s, false)) != TM_OK) return rc;
    RowsCall c;
    c.x = q->x, c.tokens = q->tokens, c.width = q->width, c.expert_rows = base + out, c.input = q->input, c.input_ld = q->input_ld, c.slots = m.slots;
    c.weights = m.weights, c.top = q->top, c.gate = q->gate, c.gate_ld = q->gate_ld, c.gate_bias = q->gate_bias, c.mult = q->mult;
    c.weight_a = q->norm_weight, c.out_a = q->norm_weight ? q->norm_out : nullptr, c.out_ld = q->input_ld, c.eps = q->norm_eps;
    return norm_rows(h, c, f32, s, false);
}
