// ---------------------------------------------------------------------------
// decoder_latent.cu -- decoder with latent attention, gated attention output, norms on
// the sublayers' outputs and a GELU-gated MLP: architecture "Maposun".
//
//   y = x + N1(attention(x)),  z = y + N2(mlp(y))        (no norm in front of a sublayer)
//
// config.json lists the layers; each names its mixer type with the mixer's sizes and
// its MLP (or none), and may use an earlier layer's tensors ("weights_of") with a cache
// of its own.  Mixer types differ in the pairing of the rotary dimensions and in whether
// the softmax has a sink (kMixerTypes); everything else is read from the configuration.
//
// How it is laid out here (latent.cuh has the two forms of latent attention):
//  * all projections that read x (query latent, key/value latent with the rotated key
//    part, gate) are one matrix; gate and up of the MLP are another;
//  * the rows of the rotated parts are permuted when the weights are packed so that a
//    pair always sits 8 rows apart (SkinnyPairRot); query and key use the same order,
//    so scores do not change, and both pairings are one code path from there on;
//  * every size is padded to a multiple of 16 with zero rows / columns;
//  * many tokens: tensor-core GEMMs, expanded keys and values, tcgen05 attention;
//    few tokens: streaming kernels and absorbed attention on the latent cache.
// A session of type B200P_F32 packs the weights as fp32 and runs everything in true fp32.
// ---------------------------------------------------------------------------
#include "session.cuh"
#include "latent.cuh"
#include "model.hpp"
#include "weights.cuh"
#include <algorithm>
#include <cmath>
#include <map>
#include <string>
#include <tuple>
#include <type_traits>

namespace b200p {
namespace {

// ---- configuration --------------------------------------------------------------------------------
struct MixerType { const char* name; bool interleaved, sink; };
const MixerType kMixerTypes[] = {
    {"latent_attention", true, false},        // pairs (2i, 2i + 1)
    {"latent_attention_2", false, true},      // pairs (i, i + dims / 2); a learned sink per head
};

struct LatentMixer {
    const MixerType* type = nullptr;
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0, q_rank = 0, rot_dims = 0;
    double rot_base = 0.0, scale = 0.0;
    int rot_pairs() const { return (rot_dim + 1) / 2; }
    LatentDims dims() const {
        return LatentDims{heads, pad16(dim), std::max(16, pad16(2 * rot_pairs())), pad16(vdim), pad16(kv_rank), pad16(q_rank)};
    }
};
struct LatentLayer {
    LatentMixer mix;
    int ff = 0;                               // 0: no MLP
    int own = 0;                              // the layer whose tensors it uses (itself, or an earlier one)
};
struct LatentSpec {
    int width = 0, vocab = 0;
    double eps = 0.0;
    std::vector<LatentLayer> layers;
};

int latent_configure(b200p_model* m, std::vector<TensorWant>* want) {
    auto spec = std::make_shared<LatentSpec>();
    const Json& c = m->config;
    const Json* layers = c.get("layers");
    if (!read_int(&c, "width", &spec->width) || !read_int(&c, "vocab", &spec->vocab) || !read_num(c.get("norm"), "eps", &spec->eps) ||
        !layers || layers->kind != Json::Array || layers->items.empty()) return B200P_E_IO;
    const long long D = spec->width, V = spec->vocab;
    want->push_back({"embed", {V, D}});
    for (size_t i = 0; i < layers->items.size(); ++i) {
        const Json& e = layers->items[i];
        LatentLayer L;
        const Json *type = e.get("type"), *mx = e.get("mixer"), *mlp = e.get("mlp"), *of = e.get("weights_of");
        if (!type || !mx) return B200P_E_IO;
        LatentMixer& x = L.mix;
        for (const MixerType& t : kMixerTypes) if (type->str == t.name) x.type = &t;
        if (!x.type) return B200P_E_OP;
        const Json* rot = mx->get("rot");
        if (!read_int(mx, "heads", &x.heads) || !read_int(mx, "dim", &x.dim) || !read_int(mx, "rot_dim", &x.rot_dim, 0) || !read_int(mx, "vdim", &x.vdim) ||
            !read_int(mx, "kv_rank", &x.kv_rank) || !read_int(mx, "q_rank", &x.q_rank) || !read_num(mx, "scale", &x.scale) ||
            !read_int(rot, "dims", &x.rot_dims, 0) || !read_num(rot, "base", &x.rot_base)) return B200P_E_IO;
        if (x.rot_dims % 2 != 0 || x.rot_dims > x.rot_dim || x.rot_base <= 0.0) return B200P_E_DIM;
        if (mlp) {
            const Json* kind = mlp->get("kind");
            if (!kind || kind->str != "dense") return B200P_E_OP;
            if (!read_int(mlp, "ff", &L.ff)) return B200P_E_IO;
        }
        L.own = int(i);
        if (of) {
            if (!of->is_int() || of->num < 0 || of->num >= double(i)) return B200P_E_IO;
            L.own = spec->layers[size_t(of->num)].own;
            const LatentLayer& o = spec->layers[size_t(L.own)];
            if (o.mix.type != x.type || o.mix.heads != x.heads || o.mix.dim != x.dim || o.mix.rot_dim != x.rot_dim || o.mix.vdim != x.vdim ||
                o.mix.kv_rank != x.kv_rank || o.mix.q_rank != x.q_rank || o.ff != L.ff) return B200P_E_DIM;
        } else {
            const long long H = x.heads, Q = x.q_rank, R = x.kv_rank, F = L.ff;
            const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
            want->push_back({p + "norm1", {D}});
            want->push_back({mp + "dq", {Q, D}});
            want->push_back({mp + "dq.norm", {Q}});
            want->push_back({mp + "uq", {H * (x.dim + x.rot_dim), Q}});
            want->push_back({mp + "dkv", {R + x.rot_dim, D}});
            want->push_back({mp + "dkv.norm", {R}});
            want->push_back({mp + "uk", {H * x.dim, R}});
            want->push_back({mp + "uv", {H * x.vdim, R}});
            if (x.type->sink) want->push_back({mp + "sink", {H}});
            want->push_back({mp + "g", {H * x.vdim, D}});
            want->push_back({mp + "o", {D, H * x.vdim}});
            if (F) {
                want->push_back({p + "norm2", {D}});
                want->push_back({p + "mlp.gate", {F, D}});
                want->push_back({p + "mlp.up", {F, D}});
                want->push_back({p + "mlp.down", {D, F}});
            }
        }
        spec->layers.push_back(L);
    }
    want->push_back({"final.norm", {D}});
    want->push_back({"head", {V, D}});
    m->w.cfg = b200p_model_config{};
    m->w.cfg.n_layers = int(spec->layers.size()); m->w.cfg.hidden = spec->width; m->w.cfg.vocab_size = spec->vocab;
    m->w.dtype = B200P_BF16;
    m->spec = spec;
    return B200P_OK;
}

// ---- packed weights -------------------------------------------------------------------------------
// The tensors of one layer, packed and padded (T elements except the sink).
struct LatentWeights {
    void *proj = nullptr, *uq = nullptr, *kv = nullptr, *ukT = nullptr, *o = nullptr, *gu = nullptr, *down = nullptr;
    void *norm1 = nullptr, *norm2 = nullptr, *q_norm = nullptr, *kv_norm = nullptr;
    float* sink = nullptr;
};

struct LatentState {
    LatentSpec spec;
    std::vector<LatentWeights> w;                      // by layer; shared layers repeat their owner's pointers
    std::vector<void*> cache;                          // by layer: [batch][max_seq][cache_row]
    std::vector<std::pair<float*, float*>> rot;        // by layer: cos, sin [max_seq][rot / 2]
    int H = 0, max_ff = 0, max_proj = 0, max_q = 0, max_qrank = 0, max_kv = 0, max_v = 0;
    // activations of the current scratch
    float *proj = nullptr, *y = nullptr, *gu = nullptr;
    void *x16 = nullptr, *cq = nullptr, *q = nullptr, *attn = nullptr, *act = nullptr;
    float *x2 = nullptr, *part_o = nullptr, *part_ml = nullptr;        // few tokens: the other residual buffer; attention's partial results
    void *q_abs = nullptr, *merged = nullptr;
    void* kv = nullptr;                                // expanded keys and values [batch][N][kv_row]
};
LatentState* latent(const b200p_session* s) { return static_cast<LatentState*>(s->decoder.get()); }

// ---- kernels: one warp per row ------------------------------------------------------------------------
// x += RMSNorm(y) * w in fp32 (y null: x as it is), and the 16-bit copy of x that the next matrix product reads.
// WPR warps of a CTA share a row: one where there are many rows, all eight in the decode step.
template <typename T, int WPR>
__global__ void __launch_bounds__(256)
postnorm_add_kernel(float* __restrict__ X, const float* __restrict__ Y, const T* __restrict__ W, T* __restrict__ X16, int rows, int H, int n, float eps) {
    griddep_launch_dependents();
    griddep_wait();
    __shared__ float part[8];
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32 + 32 * (warp % WPR);
    const int r = blockIdx.x * (8 / WPR) + warp / WPR;
    if (r >= rows) return;                                    // (WPR = 8: the whole CTA or nothing)
    float* x = X + size_t(r) * H;
    const float* y = Y ? Y + size_t(r) * H : nullptr;
    const int quads = H / 4;
    constexpr int STEP = 32 * WPR, CACHE = WPR == 1 ? 16 : 4;
    float4 c[CACHE], xv[WPR == 1 ? 1 : CACHE];                // many rows: x is read after the sum, there is enough in flight
    float ss = 0.f;
    #pragma unroll
    for (int i = 0; i < CACHE; ++i) {
        const int q = lane + STEP * i;
        if (q < quads) {
            if (WPR > 1) xv[WPR == 1 ? 0 : i] = load4<float>(x + 4 * q);
            if (y) { c[i] = load4<float>(y + 4 * q); ss += c[i].x * c[i].x + c[i].y * c[i].y + c[i].z * c[i].z + c[i].w * c[i].w; }
        }
    }
    if (y) for (int q = lane + STEP * CACHE; q < quads; q += STEP) { const float4 v = load4<float>(y + 4 * q); ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
    ss = wave::dpp::reduce_sum(ss);
    if (WPR > 1) {
        if (threadIdx.x % 32 == 0) part[warp] = ss;
        __syncthreads();
        ss = 0.f;
        #pragma unroll
        for (int k = 0; k < WPR; ++k) ss += part[k];
    }
    const float inv = rsqrtf(ss / n + eps);
    auto put = [&](int q, float4 o, const float4& v) {
        if (y) {
            const float4 w = load4<T>(W + 4 * q);
            o.x += v.x * inv * w.x; o.y += v.y * inv * w.y; o.z += v.z * inv * w.z; o.w += v.w * inv * w.w;
            store4<float>(x + 4 * q, o);
        }
        if (!std::is_same_v<T, float>) store4<T>(X16 + size_t(r) * H + 4 * q, o);
    };
    #pragma unroll
    for (int i = 0; i < CACHE; ++i) { const int q = lane + STEP * i; if (q < quads) put(q, WPR > 1 ? xv[WPR == 1 ? 0 : i] : load4<float>(x + 4 * q), c[i]); }
    for (int q = lane + STEP * CACHE; q < quads; q += STEP) put(q, load4<float>(x + 4 * q), y ? load4<float>(y + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f));
}

template <typename T>
int postnorm_add(float* x, const float* y, const void* w, void* x16, int rows, int H, int n, float eps, cudaStream_t st) {
    if (rows > 64) {
        postnorm_add_kernel<T, 1><<<blocks(size_t(rows) * 32), 256, 0, st>>>(x, y, static_cast<const T*>(w), static_cast<T*>(x16), rows, H, n, eps);
        return launched();
    }
    return launch_dependent(postnorm_add_kernel<T, 8>, dim3(unsigned(rows)), 256, 0, st, x, y, static_cast<const T*>(w), static_cast<T*>(x16), rows, H, n, eps);
}

struct LatentNormArgs {
    LatentDims d;
    const float* proj;                                 // [rows][proj_row]
    const void *q_norm, *kv_norm;
    void *cq, *cache;                                  // [rows][qrank]; [batch][max_seq][cache_row]
    const float *cos_t, *sin_t;
    int rows, Tn, pos0, max_seq, q_rank, kv_rank;      // the ranks without padding: what the means are over
    float eps;
};

// RMSNorm of n of `len` columns (the rest is padding), written as T.
template <typename T>
__device__ __forceinline__ void norm_row(const float* x, const T* w, T* y, int len, int n, float eps, int lane) {
    float ss = 0.f;
    for (int q = lane; q < len / 4; q += 32) { const float4 v = load4<float>(x + 4 * q); ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
    const float inv = rsqrtf(wave::dpp::reduce_sum(ss) / n + eps);
    for (int q = lane; q < len / 4; q += 32) {
        const float4 v = load4<float>(x + 4 * q), g = load4<T>(w + 4 * q);
        store4<T>(y + 4 * q, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
    }
}

// The two latents of a token: job 0 normalises the query latent, job 1 the key/value latent into the cache, with the
// rotated key part behind it.
template <typename T>
__global__ void __launch_bounds__(256) latent_norm_kernel(const LatentNormArgs a) {
    const int j = blockIdx.x * (blockDim.x / 32) + threadIdx.x / 32, lane = threadIdx.x % 32;
    const int r = j >> 1;
    if (r >= a.rows) return;
    const float* p = a.proj + size_t(r) * a.d.proj_row();
    if ((j & 1) == 0) {
        norm_row<T>(p, static_cast<const T*>(a.q_norm), static_cast<T*>(a.cq) + size_t(r) * a.d.qrank, a.d.qrank, a.q_rank, a.eps, lane);
        return;
    }
    const int pos = a.pos0 + r % a.Tn;
    T* row = static_cast<T*>(a.cache) + (size_t(r / a.Tn) * a.max_seq + pos) * a.d.cache_row();
    norm_row<T>(p + a.d.qrank, static_cast<const T*>(a.kv_norm), row, a.d.rank, a.kv_rank, a.eps, lane);
    const float* k = p + a.d.qrank + a.d.rank;
    for (int i = lane; i < a.d.rot / 2; i += 32) {
        const int u = 16 * (i / 8) + i % 8;
        const size_t t = size_t(pos) * (a.d.rot / 2) + i;
        const float c = a.cos_t[t], sn = a.sin_t[t], x0 = k[u], x1 = k[u + 8];
        row[a.d.rank + u] = from_float<T>(x0 * c - x1 * sn);
        row[a.d.rank + u + 8] = from_float<T>(x1 * c + x0 * sn);
    }
}

// Rotates the queries' rotated parts in place: a thread takes one group of eight pairs (16 columns) of a token and every
// kRotHeads-th head.
constexpr int kRotHeads = 8;
template <typename T>
__global__ void __launch_bounds__(256) rotate_queries_kernel(T* __restrict__ q, const float* __restrict__ cos_t, const float* __restrict__ sin_t, LatentDims d,
                                                             int rows, int Tn, int pos0) {
    const size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x;
    const int groups = d.rot / 16;
    if (i >= size_t(rows) * kRotHeads * groups) return;
    const int gr = int(i % groups), h0 = int(i / groups % kRotHeads), r = int(i / groups / kRotHeads);
    const size_t t = size_t(pos0 + r % Tn) * (d.rot / 2) + 8 * gr;
    struct alignas(16) Eight { T e[8]; };                     // 16 (fp32: 32) bytes
    const float4 c[2] = {load4<float>(cos_t + t), load4<float>(cos_t + t + 4)}, sn[2] = {load4<float>(sin_t + t), load4<float>(sin_t + t + 4)};
    const float cf[8] = {c[0].x, c[0].y, c[0].z, c[0].w, c[1].x, c[1].y, c[1].z, c[1].w};
    const float sf[8] = {sn[0].x, sn[0].y, sn[0].z, sn[0].w, sn[1].x, sn[1].y, sn[1].z, sn[1].w};
    T* v = q + size_t(r) * d.q_row() + d.dim + 16 * gr;
    #pragma unroll 2
    for (int h = h0; h < d.heads; h += kRotHeads) {
        Eight* p = reinterpret_cast<Eight*>(v + size_t(h) * (d.dim + d.rot));
        Eight a = p[0], b = p[1];
        #pragma unroll
        for (int k = 0; k < 8; ++k) {
            const float x0 = to_float(a.e[k]), x1 = to_float(b.e[k]);
            a.e[k] = from_float<T>(x0 * cf[k] - x1 * sf[k]);
            b.e[k] = from_float<T>(x1 * cf[k] + x0 * sf[k]);
        }
        p[0] = a; p[1] = b;
    }
}

template <typename T>
__global__ void gelu_mul_kernel(const float* __restrict__ gu, T* __restrict__ act, size_t M, int F) {
    const size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x;
    if (i >= M * F) return;
    const float* row = gu + i / F * 2 * F;
    act[i] = from_float<T>(gelu_tanh(row[i % F]) * row[F + i % F]);
}

// ---- many tokens, or fp32 -------------------------------------------------------------------------------
template <typename T>
int layers_gemm(b200p_session* s, int Tn, int pos0, cudaStream_t st) {
    LatentState* L = latent(s);
    constexpr bool f32 = std::is_same_v<T, float>;
    const int M = s->batch * Tn, H = L->H, n = L->spec.width, N = pos0 + Tn;
    const float eps = s->eps;
    T* xop = f32 ? reinterpret_cast<T*>(s->hidden) : static_cast<T*>(L->x16);       // what the products read
    auto add = [&](const float* y, const void* w) -> int {
        return postnorm_add<T>(s->hidden, y, w, L->x16, M, H, n, eps, st);
    };
    if (!f32) if (int e = add(nullptr, nullptr)) return e;
    for (size_t li = 0; li < L->spec.layers.size(); ++li) {
        const LatentLayer& ly = L->spec.layers[li];
        const LatentWeights& w = L->w[li];
        const LatentDims d = ly.mix.dims();
        const int qr = d.q_row(), kr = d.kv_row(), C = d.cache_row();
        T* cache = static_cast<T*>(L->cache[li]);
        // latents, rotated key part and gate; norms and the cache
        if (int e = session_gemm(s, xop, w.proj, L->proj, M, d.proj_row(), H, H, d.proj_row(), true, false, st)) return e;
        LatentNormArgs na{d, L->proj, w.q_norm, w.kv_norm, L->cq, cache, L->rot[li].first, L->rot[li].second, M, Tn, pos0, s->max_seq,
                          ly.mix.q_rank, ly.mix.kv_rank, eps};
        latent_norm_kernel<T><<<blocks(size_t(M) * 64), 256, 0, st>>>(na);
        if (int e = launched()) return e;
        // queries
        if (int e = session_gemm(s, L->cq, w.uq, L->q, M, qr, d.qrank, d.qrank, qr, f32, false, st)) return e;
        rotate_queries_kernel<T><<<blocks(size_t(M) * kRotHeads * (d.rot / 16)), 256, 0, st>>>(static_cast<T*>(L->q), L->rot[li].first, L->rot[li].second, d, M, Tn, pos0);
        if (int e = launched()) return e;
        // keys and values of everything in the cache
        for (int b = 0; b < s->batch; ++b)
            if (int e = session_gemm(s, cache + size_t(b) * s->max_seq * C, w.kv, static_cast<T*>(L->kv) + size_t(b) * N * kr, N, kr, d.rank, C, kr, f32, false, st)) return e;
        LatentAttn a{d, s->dtype, s->batch, Tn, pos0, s->max_seq, float(ly.mix.scale), w.sink, L->q, L->kv, cache, L->proj, L->attn};
        int done = f32 || tuning(KNOB_LATENT_PLAIN, 0) != 0 ? B200P_E_RANGE : latent_attn_prefill(a, st);
        if (done == B200P_E_RANGE) done = latent_attn_plain(a, st);
        if (done) return done;
        // output projection, norm, residual
        if (int e = session_gemm(s, L->attn, w.o, L->y, M, H, d.v_row(), d.v_row(), H, true, false, st)) return e;
        if (int e = add(L->y, w.norm1)) return e;
        if (!ly.ff) continue;
        const int F = pad16(ly.ff);
        int fused = B200P_E_RANGE;
        if (!f32 && tuning(KNOB_RUNTIME_GEMM, 1) != 0) {
            fused = gemm_tc(s->dtype, GEMM_EPI_GELU16, xop, w.gu, L->act, M, F, H, H, H, F, st);
            if (fused == B200P_OK) ++s->gemm_calls;
            else if (fused != B200P_E_RANGE && fused != B200P_E_ALIGN) return fused;
        }
        if (fused != B200P_OK) {
            if (int e = session_gemm(s, xop, w.gu, L->gu, M, 2 * F, H, H, 2 * F, true, false, st)) return e;
            gelu_mul_kernel<T><<<blocks(size_t(M) * F), 256, 0, st>>>(L->gu, static_cast<T*>(L->act), size_t(M), F);
            if (int e = launched()) return e;
        }
        if (int e = session_gemm(s, L->act, w.down, L->y, M, H, F, F, H, true, false, st)) return e;
        if (int e = add(L->y, w.norm2)) return e;
    }
    s->final_x = s->hidden;
    return B200P_OK;
}

// ---- few tokens -------------------------------------------------------------------------------------------
// Whether M tokens run on the streaming kernels and the absorbed attention.
bool few_tokens(const b200p_session* s, int M) {
    if (!skinny_ok(s, M) || tuning(KNOB_LATENT_PLAIN, 0) != 0) return false;
    for (const LatentLayer& l : latent(s)->spec.layers) if (!latent_step_ok(l.mix.dims(), M)) return false;
    return true;
}

// Ten launches a layer, each a programmatic dependent of the one before.  The norms on the sublayers' outputs and the
// residual adds are prologues of whatever reads x next (PRO_POSTADD: every CTA forms the sum, CTA 0 keeps it in the other
// of two buffers), so y and the norm's weights travel along as `pending`.  With more rows than kFusedAddRows every CTA
// would read too much fp32 for that: then the sum is a kernel of its own, which leaves x as 16-bit rows.
constexpr int kFusedAddRows = 4;

template <int EPI>
int launch_reading_x(SkinnyArgs& a, bool fused, cudaStream_t st) {
    using T = __nv_bfloat16;
    return fused ? launch_skinny<T, PRO_POSTADD, EPI>(a, st) : launch_skinny<T, PRO_PLAIN, EPI>(a, st);
}

int layers_few(b200p_session* s, int Tn, int pos0, cudaStream_t st, const int* pos_dev) {
    using T = __nv_bfloat16;
    LatentState* L = latent(s);
    const int M = s->batch * Tn, H = L->H, n = L->spec.width;
    float *x = s->hidden, *other = L->x2;
    const float* pending = nullptr;
    const void* pending_w = s->final_norm;              // any valid norm weights while nothing is pending
    auto args = [&](const void* W, void* out, int N, int K, int ldo) {
        SkinnyArgs a{};
        a.M = M; a.eps = s->eps; a.abort_word = s->d_abort; a.W = W; a.out = out; a.N = N; a.K = K; a.ldo = ldo;
        ++s->gemm_calls;
        return a;
    };
    const bool fused = M <= kFusedAddRows;
    auto read_x = [&](SkinnyArgs& a) {                  // X = x + norm(pending)
        if (!fused) {
            a.X16 = L->x16; a.ldx = H;
            const int e = postnorm_add<T>(x, pending, pending_w, L->x16, M, H, n, s->eps, st);
            pending = nullptr;
            return e;
        }
        a.X32 = x; a.Y32 = pending; a.x_out = other; a.norm_w = pending_w; a.norm_n = n;
        if (pending) std::swap(x, other);
        pending = nullptr;
        return int(B200P_OK);
    };
    // y = X . W^T with rows of X that may be too long for the streaming kernel's shared memory
    auto plain = [&](SkinnyArgs& a, const void* X, const void* W, int N, int K) -> int {
        a = args(W, L->y, N, K, N);
        a.X16 = X; a.ldx = K;
        const int e = launch_skinny<T, PRO_PLAIN, EPI_STORE32>(a, st);
        if (e != B200P_E_RANGE) return e;
        --s->gemm_calls;
        return session_gemm(s, X, W, L->y, M, N, K, K, N, true, false, st);
    };
    for (size_t li = 0; li < L->spec.layers.size(); ++li) {
        const LatentLayer& ly = L->spec.layers[li];
        const LatentWeights& w = L->w[li];
        const LatentDims d = ly.mix.dims();
        SkinnyArgs a = args(w.proj, L->proj, d.proj_row(), H, d.proj_row());
        if (int e = read_x(a)) return e;
        if (int e = launch_reading_x<EPI_STORE32>(a, fused, st)) return e;
        a = args(w.uq, L->q, d.q_row(), d.qrank, d.heads * d.dim);
        a.X32 = L->proj; a.ldx32 = d.proj_row(); a.norm_w = w.q_norm; a.norm_n = ly.mix.q_rank;
        a.pair = SkinnyPairRot{L->rot[li].first, L->rot[li].second, pos_dev, L->q_abs, pos0, Tn, d.dim, d.rot, d.heads, d.cache_row(), d.rank, s->max_seq};
        if (int e = launch_skinny<T, PRO_RMSNORM, EPI_PAIRROT>(a, st)) return e;
        LatentStep p{d, s->batch, Tn, pos0, s->max_seq, pos_dev, float(ly.mix.scale), s->eps, ly.mix.kv_rank, w.sink, w.ukT,
                     static_cast<const T*>(w.kv) + size_t(d.heads) * d.dim * d.rank, w.kv_norm, L->rot[li].first, L->rot[li].second,
                     L->proj, L->q, L->q_abs, L->cache[li], L->part_o, L->part_ml, L->merged, L->attn, s->d_attn_status};
        if (int e = latent_step_absorb(p, st)) return e;
        if (int e = latent_step_attend(p, st)) return e;
        if (int e = latent_step_values(p, st)) return e;
        if (int e = plain(a, L->attn, w.o, H, d.v_row())) return e;
        pending = L->y; pending_w = w.norm1;
        if (!ly.ff) continue;
        const int F = pad16(ly.ff);
        a = args(w.gu, L->act, F, H, F);
        if (int e = read_x(a)) return e;
        if (int e = launch_reading_x<EPI_GELU16>(a, fused, st)) return e;
        if (int e = plain(a, L->act, w.down, H, F)) return e;
        pending = L->y; pending_w = w.norm2;
    }
    s->final_x = x;
    return postnorm_add<T>(x, pending, pending_w, L->x16, M, H, n, s->eps, st);
}

template <typename T>
int latent_run_layers(b200p_session* s, int Tn, int pos0, cudaStream_t st, const int* pos_dev) {
    if (!std::is_same_v<T, float> && few_tokens(s, s->batch * Tn)) return layers_few(s, Tn, pos0, st, pos_dev);
    if (pos_dev) pos0 = s->kv_len;
    return layers_gemm<T>(s, Tn, pos0, st);
}

template <typename T>
int latent_alloc_scratch(b200p_session* s, int M) {
    LatentState* L = latent(s);
    const size_t m = size_t(M), e = sizeof(T);
    cudaError_t c;
    if ((c = s->alloc_scratch(&L->x16, m * L->H * e))) return int(c);
    if ((c = s->alloc_scratch(&L->proj, m * L->max_proj * 4))) return int(c);
    if ((c = s->alloc_scratch(&L->cq, m * L->max_qrank * e))) return int(c);
    if ((c = s->alloc_scratch(&L->q, m * L->max_q * e))) return int(c);
    if ((c = s->alloc_scratch(&L->attn, m * L->max_v * e))) return int(c);
    if ((c = s->alloc_scratch(&L->y, m * L->H * 4))) return int(c);
    if ((c = s->alloc_scratch(&L->act, m * L->max_ff * e))) return int(c);
    if ((c = s->alloc_scratch(&L->x2, std::min<size_t>(m, kSkinnyMaxM) * L->H * 4))) return int(c);
    if ((c = s->alloc_scratch(&L->gu, m * 2 * L->max_ff * 4))) return int(c);
    return B200P_OK;
}

bool latent_graph_step(const b200p_session* s) { return few_tokens(s, s->batch); }
int latent_gemms_per_step(const b200p_session* s) {
    int n = 0;
    for (const LatentLayer& l : latent(s)->spec.layers) n += l.ff ? 5 : 3;
    return n;
}

// ---- session -------------------------------------------------------------------------------------------
template <typename T>
int build_weights(b200p_session* s, const b200p_model* m) {
    LatentState* L = latent(s);
    const LatentSpec& spec = L->spec;
    const int H = L->H;
    WeightPacker<T> pk{s, m};
    int& rc = pk.rc;
    auto zeros = [&](size_t n, size_t esz) { return pk.zeros(n, esz); };
    auto put = [&](void* dst, const std::string& name, const Where& row_at, const Where& col_at) { pk.put(dst, name, row_at, col_at); };
    auto padded = [&](const std::string& name, int rows_p, int ld) { return pk.padded(name, rows_p, ld); };
    const Where same = at_index();
    auto stride = [](long long ld, long long first = 0) { return at_stride(ld, first); };
    s->embed = padded("embed", spec.vocab, H);
    s->lm_head = padded("head", spec.vocab, H);
    s->final_norm = padded("final.norm", 1, H);
    L->w.resize(spec.layers.size());
    for (size_t i = 0; i < spec.layers.size() && !rc; ++i) {
        const LatentLayer& ly = spec.layers[i];
        if (ly.own != int(i)) { L->w[i] = L->w[size_t(ly.own)]; continue; }
        LatentWeights& w = L->w[i];
        const LatentMixer& x = ly.mix;
        const LatentDims d = x.dims();
        const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
        // dimension j of a rotated part -> its place: pairs 8 apart, in groups of 16; dimensions past rot_dims, which
        // pass unrotated, are further pairs with angle 0
        auto rot_at = [x](int j) -> int {
            int pair, second;
            if (j >= x.rot_dims)          { pair = x.rot_dims / 2 + (j - x.rot_dims) / 2; second = (j - x.rot_dims) % 2; }
            else if (x.type->interleaved) { pair = j / 2; second = j % 2; }
            else                          { pair = j % (x.rot_dims / 2); second = j >= x.rot_dims / 2; }
            return 16 * (pair / 8) + pair % 8 + 8 * second;
        };
        auto by_head = [](int n, int np) { return [=](int r) -> long long { return (long long)(r / n) * np + r % n; }; };
        const auto v_at = by_head(x.vdim, d.vdim), k_at = by_head(x.dim, d.dim);
        w.norm1 = padded(p + "norm1", 1, H);
        w.q_norm = padded(mp + "dq.norm", 1, d.qrank);
        w.kv_norm = padded(mp + "dkv.norm", 1, d.rank);
        w.proj = zeros(size_t(d.proj_row()) * H, sizeof(T));
        put(w.proj, mp + "dq", stride(H), same);
        put(w.proj, mp + "dkv", [=](int r) { return (long long)(d.qrank + (r < x.kv_rank ? r : d.rank + rot_at(r - x.kv_rank))) * H; }, same);
        put(w.proj, mp + "g", [=](int r) { return (d.gate_col() + v_at(r)) * H; }, same);
        w.uq = zeros(size_t(d.q_row()) * d.qrank, sizeof(T));
        put(w.uq, mp + "uq", [=](int r) {
            const int h = r / (x.dim + x.rot_dim), j = r % (x.dim + x.rot_dim);
            return ((long long)h * (d.dim + d.rot) + (j < x.dim ? j : d.dim + rot_at(j - x.dim))) * d.qrank;
        }, same);
        w.kv = zeros(size_t(d.kv_row()) * d.rank, sizeof(T));
        put(w.kv, mp + "uk", [=](int r) { return k_at(r) * d.rank; }, same);
        put(w.kv, mp + "uv", [=](int r) { return ((long long)d.heads * d.dim + v_at(r)) * d.rank; }, same);
        w.ukT = zeros(size_t(d.heads) * d.rank * d.dim, sizeof(T));                 // [head][rank][dim]
        put(w.ukT, mp + "uk", [=](int r) { return (long long)(r / x.dim) * d.rank * d.dim + r % x.dim; }, stride(d.dim));
        if (d.vdim == x.vdim) w.o = padded(mp + "o", H, d.v_row());
        else {
            w.o = zeros(size_t(H) * d.v_row(), sizeof(T));
            put(w.o, mp + "o", stride(d.v_row()), v_at);
        }
        if (x.type->sink) {
            w.sink = static_cast<float*>(zeros(size_t(d.heads), 4));
            if (!rc) rc = pack<float>(w.sink, m->tensors.at(mp + "sink"), same, same);
        }
        if (ly.ff) {
            const int F = pad16(ly.ff);
            w.norm2 = padded(p + "norm2", 1, H);
            w.gu = zeros(size_t(2) * F * H, sizeof(T));
            put(w.gu, p + "mlp.gate", stride(H), same);
            put(w.gu, p + "mlp.up", stride(H, F), same);
            w.down = padded(p + "mlp.down", H, F);
        }
    }
    return rc;
}

// Angles p * base^(-2i / dims), [max_seq][rot / 2]; pairs past dims / 2 do not turn.
int build_rotation(b200p_session* s, const LatentMixer& x, std::pair<float*, float*>* out) {
    std::vector<double> f;
    for (int i = 0; i < x.rot_dims / 2; ++i) f.push_back(std::pow(x.rot_base, -2.0 * i / x.rot_dims));
    return rotation_table(s, f, x.dims().rot / 2, out);
}

template <typename T> const DecoderOps* latent_ops() {
    static const DecoderOps ops{latent_alloc_scratch<T>, latent_run_layers<T>, true, latent_graph_step, latent_gemms_per_step, nullptr};
    return &ops;
}

int latent_build(b200p_session* s, const b200p_model* m) {
    if (s->dtype != B200P_BF16 && s->dtype != B200P_F32) return B200P_E_DTYPE;
    auto L = std::make_shared<LatentState>();
    L->spec = *std::static_pointer_cast<LatentSpec>(m->spec);
    s->decoder = L;
    s->ops = s->dtype == B200P_F32 ? latent_ops<float>() : latent_ops<__nv_bfloat16>();
    s->H = L->H = pad16(L->spec.width);
    s->eps = float(L->spec.eps);
    if (int rc = s->dtype == B200P_F32 ? build_weights<float>(s, m) : build_weights<__nv_bfloat16>(s, m)) return rc;
    const size_t esz = s->dtype == B200P_F32 ? 4 : 2;
    std::map<std::tuple<double, int, int>, std::pair<float*, float*>> tables;
    int max_k = L->H;
    for (const LatentLayer& ly : L->spec.layers) {
        const LatentDims d = ly.mix.dims();
        L->max_ff = std::max(L->max_ff, pad16(ly.ff)); L->max_proj = std::max(L->max_proj, d.proj_row());
        L->max_q = std::max(L->max_q, d.q_row()); L->max_qrank = std::max(L->max_qrank, d.qrank);
        L->max_kv = std::max(L->max_kv, d.kv_row()); L->max_v = std::max(L->max_v, d.v_row());
        max_k = std::max(max_k, d.qrank);
        const auto key = std::make_tuple(ly.mix.rot_base, ly.mix.rot_dims, d.rot);
        if (!tables.count(key)) if (int rc = build_rotation(s, ly.mix, &tables[key])) return rc;
        L->rot.push_back(tables[key]);
        void* cache = nullptr;
        const size_t bytes = size_t(s->batch) * s->max_seq * d.cache_row() * esz;
        if (cudaError_t e = s->alloc(&cache, bytes)) return int(e);
        if (cudaError_t e = cudaMemset(cache, 0, bytes)) return int(e);
        L->cache.push_back(cache);
    }
    s->skinny_max_k = max_k;
    s->skinny_usable = s->dtype != B200P_F32;
    if (cudaError_t e = s->alloc(&L->kv, size_t(s->batch) * s->max_seq * L->max_kv * esz)) return int(e);
    if (s->dtype == B200P_BF16) {                         // the absorbed attention's queries and partial results
        size_t parts = 0, part_floats = 0, abs = 0;
        for (const LatentLayer& ly : L->spec.layers) {
            const LatentDims d = ly.mix.dims();
            const size_t n = latent_step_partials(d);
            parts = std::max(parts, n); part_floats = std::max(part_floats, n * d.rank);
            abs = std::max(abs, size_t(kSkinnyMaxM) * d.heads * d.cache_row());
        }
        if (cudaError_t e = s->alloc(&L->part_o, part_floats * 4)) return int(e);
        if (cudaError_t e = s->alloc(&L->part_ml, parts * 8)) return int(e);
        if (cudaError_t e = s->alloc(&L->q_abs, abs * 2)) return int(e);
        if (cudaError_t e = s->alloc(&L->merged, abs * 2)) return int(e);
    }
    if (cudaError_t e = s->alloc(&s->d_attn_status, 16)) return int(e);
    return int(cudaMemset(s->d_attn_status, 0, 16));
}

const ArchitectureEntry entry("Maposun", latent_configure, latent_build);

} // namespace
} // namespace b200p
