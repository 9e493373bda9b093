// ---------------------------------------------------------------------------
// decoder_hybrid.cu -- decoder whose layers mix the gated delta rule with attention under a
// window or in chunks, pre-norm, SiLU MLP or none, a span of layers that runs several times:
// architecture "Vofusun".
//
//   x = scale * embedding;   y = x + mixer(N1(x)),  z = y + mlp(N2(y));   logits = embedding . N(z)
//
// config.json lists the layers; each names its mixer type with the mixer's sizes and its MLP
// (or none).  "loop" names the span that runs `times` times with the same tensors; every run
// of a layer (a pass) has a cache or state of its own, and ahead of every pass of the span but
// the first the embeddings are added to x once more.  What tells the mixer types apart is in
// kMixerTypes; everything else is read from the configuration.
//
// How it is laid out here (grouped_attn.cuh, delta.cuh):
//  * all projections that read the normalised x are one matrix; gate and up of the MLP are
//    another; the inputs of decays and step sizes are the first matrix's last rows, whose
//    products stay fp32;
//  * every size is padded to a multiple of 16 with zero rows / columns;
//  * prompts: tensor-core GEMMs, the residual sum in their epilogue, tcgen05 attention, the
//    delta rule in blocks;
//  * one new token per sequence (up to 16): five launches a layer, norms as prologues and
//    SiLU / residual sum as epilogues of the streaming projections, the mixer from projection
//    to gated output in one kernel.
// A session of type B200P_F32 packs the weights as fp32 and runs everything in true fp32.
// ---------------------------------------------------------------------------
#include "session.cuh"
#include "delta.cuh"
#include "grouped_attn.cuh"
#include "model.hpp"
#include "weights.cuh"
#include <algorithm>
#include <cmath>
#include <map>
#include <string>
#include <type_traits>

namespace b200p {
namespace {

// ---- configuration --------------------------------------------------------------------------------
struct MixerType {
    const char* name;
    bool delta;                               // gated delta rule; the rest describes attention
    int mask;                                 // AttnMaskKind
    bool rotated, normed, own_values, gated, plus_one;
};
const MixerType kMixerTypes[] = {
    {"delta", true, 0, false, false, false, false, false},
    {"attention", false, MASK_WINDOW, false, false, true, false, true},
    {"attention_2", false, MASK_CHUNK, true, true, false, true, true},      // values: the keys as projected
};

struct HybridLayer {
    const MixerType* type = nullptr;
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 0, mask_size = 0;
    double scale = 0.0;
    std::vector<double> freq;                 // rotary angle per position of pair i
    int ff = 0;                               // 0: no MLP
    GroupedDims grouped() const { return GroupedDims{heads, kv_heads, pad16(dim), pad16(vdim), dim, type->own_values, type->gated}; }
    DeltaDims delta() const { return DeltaDims{heads, kv_heads, pad16(dim), pad16(vdim), dim, vdim, taps}; }
    int main_row() const { return type->delta ? delta().main_row() : grouped().proj_row(); }
    int ab_row() const { return type->delta ? delta().ab_row() : 0; }
    int v_row() const { return heads * pad16(vdim); }
};
struct HybridSpec {
    int width = 0, vocab = 0;
    double eps = 0.0, embed_scale = 1.0;
    std::vector<HybridLayer> layers;
    struct Pass { int layer; bool embed_again; };
    std::vector<Pass> passes;                 // in the order they run
};

// f_i = base^(-2i / dims).  With `scaling`, frequencies that turn less than `low` times within `original` positions are
// divided by `factor`, those that turn more than `high` times stay, with a linear ramp in between.
bool read_frequencies(const Json* rot, int dim, std::vector<double>* out) {
    int dims = 0;
    double base = 0.0;
    if (!read_int(rot, "dims", &dims, 0) || !read_num(rot, "base", &base) || dims % 2 != 0 || dims > dim || base <= 0.0) return false;
    const Json* sc = rot->get("scaling");
    double factor = 1.0, low = 0.0, high = 0.0, original = 0.0;
    if (sc && (!read_num(sc, "factor", &factor) || !read_num(sc, "low", &low) || !read_num(sc, "high", &high) || !read_num(sc, "original", &original) ||
               factor <= 0.0 || original <= 0.0 || low <= 0.0 || high < low)) return false;
    for (int i = 0; i < dims / 2; ++i) {
        double f = std::pow(base, -2.0 * i / dims);
        if (sc) {
            const double turns = original * f / (2.0 * 3.14159265358979323846);
            if (turns < low) f /= factor;
            else if (turns <= high) {
                const double s = high > low ? (turns - low) / (high - low) : 1.0;
                f = (1.0 - s) * f / factor + s * f;
            }
        }
        out->push_back(f);
    }
    return true;
}

int hybrid_configure(b200p_model* m, std::vector<TensorWant>* want) {
    auto spec = std::make_shared<HybridSpec>();
    const Json& c = m->config;
    const Json *layers = c.get("layers"), *emb = c.get("embedding"), *loop = c.get("loop");
    if (!read_int(&c, "width", &spec->width) || !read_int(&c, "vocab", &spec->vocab) || !read_num(c.get("norm"), "eps", &spec->eps) ||
        (emb && emb->get("scale") && !read_num(emb, "scale", &spec->embed_scale)) || !layers || layers->kind != Json::Array || layers->items.empty()) return B200P_E_IO;
    const long long D = spec->width, V = spec->vocab;
    const int n = int(layers->items.size());
    want->push_back({"embed", {V, D}});
    for (int i = 0; i < n; ++i) {
        const Json& e = layers->items[size_t(i)];
        HybridLayer L;
        const Json *type = e.get("type"), *mx = e.get("mixer"), *mlp = e.get("mlp");
        if (!type || !mx) return B200P_E_IO;
        for (const MixerType& t : kMixerTypes) if (type->str == t.name) L.type = &t;
        if (!L.type) return B200P_E_OP;
        if (!read_int(mx, "heads", &L.heads) || !read_int(mx, "kv_heads", &L.kv_heads) || !read_int(mx, "dim", &L.dim) || !read_int(mx, "vdim", &L.vdim)) return B200P_E_IO;
        if (L.heads % L.kv_heads != 0 || L.dim > 512 || L.vdim > 512) return B200P_E_DIM;
        if (L.type->delta) {
            if (!read_int(mx, "conv", &L.taps)) return B200P_E_IO;
        } else {
            if (!read_num(mx, "scale", &L.scale) || !read_int(mx->get("mask"), "size", &L.mask_size)) return B200P_E_IO;
            if (!L.type->own_values && L.vdim != L.dim) return B200P_E_DIM;
            if (L.type->rotated && !read_frequencies(mx->get("rot"), L.dim, &L.freq)) return B200P_E_IO;
        }
        if (mlp) {
            const Json* kind = mlp->get("kind");
            if (!kind || kind->str != "dense") return B200P_E_OP;
            if (!read_int(mlp, "ff", &L.ff)) return B200P_E_IO;
        }
        const long long H = L.heads, G = L.kv_heads, d = L.dim, e_ = L.vdim, F = L.ff;
        const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
        want->push_back({p + "norm1", {D}});
        if (L.type->delta) {
            for (const char* t : {"q", "k", "v"}) {
                const long long rows = t[0] == 'v' ? H * e_ : G * d;
                want->push_back({mp + t, {rows, D}});
                want->push_back({mp + t + ".conv", {rows, L.taps}});
            }
            want->push_back({mp + "a", {H, D}});
            want->push_back({mp + "b", {H, D}});
            want->push_back({mp + "A_log", {H}});
            want->push_back({mp + "dt_bias", {H}});
            want->push_back({mp + "norm", {e_}});
        } else {
            want->push_back({mp + "q", {H * d, D}});
            want->push_back({mp + "k", {G * d, D}});
            if (L.type->own_values) want->push_back({mp + "v", {G * e_, D}});
        }
        if (L.type->delta || L.type->gated) want->push_back({mp + "g", {H * e_, D}});
        want->push_back({mp + "o", {D, H * e_}});
        if (F) {
            want->push_back({p + "norm2", {D}});
            want->push_back({p + "mlp.gate", {F, D}});
            want->push_back({p + "mlp.up", {F, D}});
            want->push_back({p + "mlp.down", {D, F}});
        }
        spec->layers.push_back(L);
    }
    int start = 0, stop = 0, times = 1;
    if (loop && (!read_int(loop, "start", &start, 0) || !read_int(loop, "stop", &stop, 0) || !read_int(loop, "times", &times) || start > stop || stop > n || times > 4096)) return B200P_E_IO;
    for (int i = 0; i < start; ++i) spec->passes.push_back({i, false});
    for (int t = 0; t < times; ++t)
        for (int i = start; i < stop; ++i) spec->passes.push_back({i, t > 0 && i == start});
    for (int i = stop; i < n; ++i) spec->passes.push_back({i, false});
    want->push_back({"final.norm", {D}});
    m->w.cfg = b200p_model_config{};
    m->w.cfg.n_layers = n; m->w.cfg.hidden = spec->width; m->w.cfg.vocab_size = spec->vocab;
    m->w.dtype = B200P_BF16;
    m->spec = spec;
    return B200P_OK;
}

// ---- state of a session -----------------------------------------------------------------------------
// The tensors of one layer, packed and padded (T elements except where noted).
struct HybridWeights {
    void *proj = nullptr, *o = nullptr, *gu = nullptr, *down = nullptr, *norm1 = nullptr, *norm2 = nullptr;
    float *conv = nullptr, *a_log = nullptr, *dt_bias = nullptr, *head_norm = nullptr;
    std::pair<float*, float*> rot{nullptr, nullptr};   // cos, sin [max_seq][dim / 2]
};
// What a pass keeps of the sequences: keys and values, or the recurrent state and the convolutions' inputs.
struct PassState { void *k = nullptr, *v = nullptr; float *state = nullptr, *ring = nullptr; };

struct HybridState {
    HybridSpec spec;
    std::vector<HybridWeights> w;                      // by layer
    std::vector<PassState> kept;                       // by pass
    int H = 0, max_ff = 0, max_main = 0, max_ab = 0, max_v = 0;
    bool looped = false;
    // activations of the current scratch
    void *norm = nullptr, *proj = nullptr, *attn = nullptr, *act = nullptr;
    float *ab = nullptr, *proj32 = nullptr, *gu = nullptr, *rows = nullptr, *cols = nullptr, *o = nullptr;
};
HybridState* hybrid(const b200p_session* s) { return static_cast<HybridState*>(s->decoder.get()); }

// ---- kernels ------------------------------------------------------------------------------------------
// x += y, n a multiple of 4
__global__ void __launch_bounds__(256) add_kernel(float* __restrict__ x, const float* __restrict__ y, size_t n) {
    griddep_launch_dependents();
    griddep_wait();
    const size_t i = (size_t(blockIdx.x) * blockDim.x + threadIdx.x) * 4;
    if (i >= n) return;
    const float4 a = load4<float>(x + i), b = load4<float>(y + i);
    store4<float>(x + i, make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w));
}

int embed_again(b200p_session* s, int M, cudaStream_t st) {
    const size_t n = size_t(M) * s->H;
    return launch_dependent(add_kernel, dim3(blocks(n / 4)), 256, 0, st, s->hidden, static_cast<const float*>(s->embedded), n);
}

GroupedAttn grouped_args(const b200p_session* s, size_t pass, int Tn, int pos0, const int* pos_dev) {
    const HybridState* L = hybrid(s);
    const HybridLayer& ly = L->spec.layers[size_t(L->spec.passes[pass].layer)];
    const HybridWeights& w = L->w[size_t(L->spec.passes[pass].layer)];
    GroupedAttn a{};
    a.d = ly.grouped();
    a.mask = AttnMask{ly.type->mask, ly.mask_size};
    a.dtype = s->dtype; a.batch = s->batch; a.Tn = Tn; a.pos0 = pos0; a.max_seq = s->max_seq; a.pos_dev = pos_dev;
    a.scale = float(ly.scale); a.eps = s->eps; a.norm = ly.type->normed; a.plus_one = ly.type->plus_one;
    a.cos_t = w.rot.first; a.sin_t = w.rot.second;
    a.proj = L->proj; a.kcache = L->kept[pass].k; a.vcache = L->kept[pass].v; a.out = L->attn;
    a.abort_word = s->d_attn_status;
    return a;
}

DeltaArgs delta_args(const b200p_session* s, size_t pass, int Tn, int pos0, const int* pos_dev) {
    const HybridState* L = hybrid(s);
    const HybridLayer& ly = L->spec.layers[size_t(L->spec.passes[pass].layer)];
    const HybridWeights& w = L->w[size_t(L->spec.passes[pass].layer)];
    DeltaArgs a{};
    a.d = ly.delta();
    a.dtype = a.proj_dtype = s->dtype; a.batch = s->batch; a.Tn = Tn; a.pos0 = pos0; a.max_seq = s->max_seq; a.pos_dev = pos_dev;
    a.eps = s->eps; a.proj = L->proj; a.ldp = a.d.main_row(); a.ab = L->ab; a.ld_ab = a.d.ab_row();
    a.conv = w.conv; a.a_log = w.a_log; a.dt_bias = w.dt_bias; a.norm = w.head_norm;
    a.state = L->kept[pass].state; a.ring = L->kept[pass].ring;
    a.rows = L->rows; a.cols = L->cols; a.o = L->o; a.out = L->attn;
    a.abort_word = s->d_attn_status;
    return a;
}

// ---- many tokens, or fp32 -------------------------------------------------------------------------------
template <typename T>
int layers_gemm(b200p_session* s, int Tn, int pos0, cudaStream_t st) {
    HybridState* L = hybrid(s);
    constexpr bool f32 = std::is_same_v<T, float>;
    const int M = s->batch * Tn, H = L->H, n = L->spec.width;
    auto normed = [&](const void* w) -> int {
        rmsnorm_cast_kernel<T><<<blocks(size_t(M) * 32), 256, 0, st>>>(s->hidden, static_cast<const T*>(w), static_cast<T*>(L->norm), M, H, n, s->eps, 1, 0);
        return launched();
    };
    s->final_x = s->hidden;
    for (size_t p = 0; p < L->spec.passes.size(); ++p) {
        const int li = L->spec.passes[p].layer;
        const HybridLayer& ly = L->spec.layers[size_t(li)];
        const HybridWeights& w = L->w[size_t(li)];
        if (L->spec.passes[p].embed_again) if (int e = embed_again(s, M, st)) return e;
        if (int e = normed(w.norm1)) return e;
        const int rows = ly.main_row();
        if (int e = session_gemm(s, L->norm, w.proj, L->proj, M, rows, H, H, rows, f32, false, st)) return e;
        if (ly.type->delta) {
            if (int e = session_gemm(s, L->norm, static_cast<const T*>(w.proj) + size_t(rows) * H, L->ab, M, ly.ab_row(), H, H, ly.ab_row(), true, false, st)) return e;
            const DeltaArgs a = delta_args(s, p, Tn, pos0, nullptr);
            int done = Tn == 1 && tuning(KNOB_DELTA_PLAIN, 0) == 0 ? delta_step(a, st) : B200P_E_RANGE;
            if (done == B200P_E_RANGE) done = delta_tokens(a, st);
            if (done) return done;
        } else {
            const GroupedAttn a = grouped_args(s, p, Tn, pos0, nullptr);
            if (int e = grouped_inputs(a, st)) return e;
            int done = f32 || tuning(KNOB_GROUPED_PLAIN, 0) != 0 ? B200P_E_RANGE : grouped_prefill(a, st);
            if (done == B200P_E_RANGE) done = grouped_plain(a, st);
            if (done) return done;
        }
        if (int e = session_gemm(s, L->attn, w.o, s->hidden, M, H, ly.v_row(), ly.v_row(), H, true, true, st)) return e;
        if (!ly.ff) continue;
        const int F = pad16(ly.ff);
        if (int e = normed(w.norm2)) return e;
        int fused = B200P_E_RANGE;
        if (!f32 && tuning(KNOB_RUNTIME_GEMM, 1) != 0) {
            fused = gemm_tc(s->dtype, GEMM_EPI_SILU16, L->norm, w.gu, L->act, M, F, H, H, H, F, st);
            if (fused == B200P_OK) ++s->gemm_calls;
            else if (fused != B200P_E_RANGE && fused != B200P_E_ALIGN) return fused;
        }
        if (fused != B200P_OK) {
            if (int e = session_gemm(s, L->norm, w.gu, L->gu, M, 2 * F, H, H, 2 * F, true, false, st)) return e;
            silu_mul_cast_kernel<T><<<blocks(size_t(M) * F), 256, 0, st>>>(L->gu, static_cast<T*>(L->act), size_t(M), F);
            if (int e = launched()) return e;
        }
        if (int e = session_gemm(s, L->act, w.down, s->hidden, M, H, F, F, H, true, true, st)) return e;
    }
    return B200P_OK;
}

// ---- one new token per sequence ---------------------------------------------------------------------------
bool step_ok(const b200p_session* s, int M) {
    if (!skinny_ok(s, M) || tuning(KNOB_GROUPED_PLAIN, 0) != 0 || tuning(KNOB_DELTA_PLAIN, 0) != 0) return false;
    for (const HybridLayer& l : hybrid(s)->spec.layers)
        if (l.type->delta ? !delta_step_ok(l.delta()) : !grouped_step_ok(l.grouped())) return false;
    return true;
}

// Five launches a layer, each a programmatic dependent of the one before.
int layers_step(b200p_session* s, int pos0, cudaStream_t st, const int* pos_dev) {
    using T = __nv_bfloat16;
    HybridState* L = hybrid(s);
    const int M = s->batch, H = L->H;
    auto args = [&](const void* W, void* out, int N, int K, int ldo) {
        SkinnyArgs a{};
        a.M = M; a.eps = s->eps; a.abort_word = s->d_abort; a.norm_n = L->spec.width; a.W = W; a.out = out; a.N = N; a.K = K; a.ldo = ldo;
        ++s->gemm_calls;
        return a;
    };
    // x += X . W^T with rows of X that may be too long for the streaming kernel's shared memory
    auto add = [&](const void* X, const void* W, int K) -> int {
        SkinnyArgs a = args(W, s->hidden, H, K, H);
        a.X16 = X; a.ldx = K;
        const int e = launch_skinny<T, PRO_PLAIN, EPI_ACC32>(a, st);
        if (e != B200P_E_RANGE) return e;
        --s->gemm_calls;
        return session_gemm(s, X, W, s->hidden, M, H, K, K, H, true, true, st);
    };
    s->final_x = s->hidden;
    for (size_t p = 0; p < L->spec.passes.size(); ++p) {
        const int li = L->spec.passes[p].layer;
        const HybridLayer& ly = L->spec.layers[size_t(li)];
        const HybridWeights& w = L->w[size_t(li)];
        if (L->spec.passes[p].embed_again) if (int e = embed_again(s, M, st)) return e;
        const int rows = ly.main_row() + ly.ab_row();
        SkinnyArgs a = args(w.proj, L->proj32, rows, H, rows);
        a.X32 = s->hidden; a.norm_w = w.norm1;
        if (int e = launch_skinny<T, PRO_RMSNORM, EPI_STORE32>(a, st)) return e;
        if (ly.type->delta) {
            DeltaArgs d = delta_args(s, p, 1, pos0, pos_dev);
            d.proj = L->proj32; d.proj_dtype = B200P_F32; d.ldp = d.ld_ab = rows; d.ab = L->proj32 + ly.main_row();
            if (int e = delta_step(d, st)) return e;
        } else {
            GroupedAttn g = grouped_args(s, p, 1, pos0, pos_dev);
            g.proj = L->proj32;
            if (int e = grouped_step(g, st)) return e;
        }
        if (int e = add(L->attn, w.o, ly.v_row())) return e;
        if (!ly.ff) continue;
        const int F = pad16(ly.ff);
        a = args(w.gu, L->act, F, H, F);
        a.X32 = s->hidden; a.norm_w = w.norm2;
        if (int e = launch_skinny<T, PRO_RMSNORM, EPI_SILU16>(a, st)) return e;
        if (int e = add(L->act, w.down, F)) return e;
    }
    return B200P_OK;
}

template <typename T>
int hybrid_run_layers(b200p_session* s, int Tn, int pos0, cudaStream_t st, const int* pos_dev) {
    if (!std::is_same_v<T, float> && Tn == 1 && step_ok(s, s->batch)) return layers_step(s, pos0, st, pos_dev);
    if (pos_dev) pos0 = s->kv_len;
    return layers_gemm<T>(s, Tn, pos0, st);
}

template <typename T>
int hybrid_alloc_scratch(b200p_session* s, int M) {
    HybridState* L = hybrid(s);
    const size_t m = size_t(M), e = sizeof(T);
    cudaError_t c;
    if ((c = s->alloc_scratch(&L->norm, m * L->H * e))) return int(c);
    if ((c = s->alloc_scratch(&L->proj, m * L->max_main * e))) return int(c);
    if ((c = s->alloc_scratch(&L->ab, m * L->max_ab * 4))) return int(c);
    if ((c = s->alloc_scratch(&L->proj32, std::min<size_t>(m, kSkinnyMaxM) * (L->max_main + L->max_ab) * 4))) return int(c);
    if ((c = s->alloc_scratch(&L->attn, m * L->max_v * e))) return int(c);
    if ((c = s->alloc_scratch(&L->act, m * L->max_ff * e))) return int(c);
    if ((c = s->alloc_scratch(&L->gu, m * 2 * L->max_ff * 4))) return int(c);
    if (L->looped) if ((c = s->alloc_scratch(&s->embedded, m * L->H * 4))) return int(c);
    DeltaScratch n{0, 0, 0};
    for (const HybridLayer& l : L->spec.layers)
        if (l.type->delta) {
            const DeltaScratch x = delta_scratch(l.delta(), s->batch, M);
            n = {std::max(n.rows, x.rows), std::max(n.cols, x.cols), std::max(n.o, x.o)};
        }
    if ((c = s->alloc_scratch(&L->rows, n.rows * 4)) || (c = s->alloc_scratch(&L->cols, n.cols * 4)) || (c = s->alloc_scratch(&L->o, n.o * 4))) return int(c);
    return B200P_OK;
}

bool hybrid_graph_step(const b200p_session* s) { return s->dtype != B200P_F32 && step_ok(s, s->batch); }
int hybrid_gemms_per_step(const b200p_session* s) {
    int n = 0;
    for (const HybridSpec::Pass& p : hybrid(s)->spec.passes) n += hybrid(s)->spec.layers[size_t(p.layer)].ff ? 4 : 2;
    return n;
}

// ---- session -------------------------------------------------------------------------------------------
template <typename T>
int build_weights(b200p_session* s, const b200p_model* m) {
    HybridState* L = hybrid(s);
    const HybridSpec& spec = L->spec;
    const int H = L->H;
    WeightPacker<T> pk{s, m};
    const Where same = at_index();
    auto f32_vector = [&](const std::string& name, int n) {
        float* p = static_cast<float*>(pk.zeros(size_t(n), 4));
        pk.put_f32(p, name, same, same);
        return p;
    };
    s->embed = s->lm_head = pk.padded("embed", spec.vocab, H);
    s->final_norm = pk.padded("final.norm", 1, H);
    L->w.resize(spec.layers.size());
    for (size_t i = 0; i < spec.layers.size() && !pk.rc; ++i) {
        const HybridLayer& ly = spec.layers[i];
        HybridWeights& w = L->w[i];
        const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
        const int d = pad16(ly.dim), e = pad16(ly.vdim), G = ly.kv_heads;
        w.norm1 = pk.padded(p + "norm1", 1, H);
        w.proj = pk.zeros(size_t(ly.main_row() + ly.ab_row()) * H, sizeof(T));
        pk.put(w.proj, mp + "q", at_heads(ly.dim, d, H), same);
        if (ly.type->delta) {
            const DeltaDims dd = ly.delta();
            const long long k0 = (long long)G * d, v0 = 2 * k0, C = dd.channels();
            pk.put(w.proj, mp + "k", at_heads(ly.dim, d, H, k0), same);
            pk.put(w.proj, mp + "v", at_heads(ly.vdim, e, H, v0), same);
            pk.put(w.proj, mp + "g", at_heads(ly.vdim, e, H, dd.g_col()), same);
            pk.put(w.proj, mp + "a", at_stride(H, ly.main_row()), same);
            pk.put(w.proj, mp + "b", at_stride(H, ly.main_row() + ly.heads), same);
            w.conv = static_cast<float*>(pk.zeros(size_t(ly.taps) * C, 4));
            pk.put_f32(w.conv, mp + "q.conv", at_heads(ly.dim, d), at_stride(C));
            pk.put_f32(w.conv, mp + "k.conv", at_heads(ly.dim, d, 1, k0), at_stride(C));
            pk.put_f32(w.conv, mp + "v.conv", at_heads(ly.vdim, e, 1, v0), at_stride(C));
            w.a_log = f32_vector(mp + "A_log", ly.heads);
            w.dt_bias = f32_vector(mp + "dt_bias", ly.heads);
            w.head_norm = f32_vector(mp + "norm", e);
        } else {
            const GroupedDims gd = ly.grouped();
            pk.put(w.proj, mp + "k", at_heads(ly.dim, d, H, gd.k_col()), same);
            if (gd.own_values) pk.put(w.proj, mp + "v", at_heads(ly.vdim, e, H, gd.v_col()), same);
            if (gd.gated) pk.put(w.proj, mp + "g", at_heads(ly.vdim, e, H, gd.g_col()), same);
            if (!pk.rc && ly.type->rotated) pk.rc = rotation_table(s, ly.freq, d / 2, &w.rot);
        }
        if (e == ly.vdim) w.o = pk.padded(mp + "o", H, ly.v_row());
        else {
            w.o = pk.zeros(size_t(H) * ly.v_row(), sizeof(T));
            pk.put(w.o, mp + "o", at_stride(ly.v_row()), at_heads(ly.vdim, e));
        }
        if (ly.ff) {
            const int F = pad16(ly.ff);
            w.norm2 = pk.padded(p + "norm2", 1, H);
            w.gu = pk.zeros(size_t(2) * F * H, sizeof(T));
            pk.put(w.gu, p + "mlp.gate", at_stride(H), same);
            pk.put(w.gu, p + "mlp.up", at_stride(H, F), same);
            w.down = pk.padded(p + "mlp.down", H, F);
        }
    }
    if (pk.rc) return pk.rc;
    const size_t rows = size_t(s->batch) * s->max_seq;
    for (const HybridSpec::Pass& pass : spec.passes) {
        const HybridLayer& ly = spec.layers[size_t(pass.layer)];
        PassState k;
        if (ly.type->delta) {
            const DeltaDims dd = ly.delta();
            k.state = static_cast<float*>(pk.zeros(size_t(s->batch) * dd.state_floats(), 4));
            k.ring = static_cast<float*>(pk.zeros(size_t(s->batch) * dd.taps * dd.channels(), 4));
        } else {
            const GroupedDims gd = ly.grouped();
            k.k = pk.zeros(rows * gd.kv_heads * gd.dim, sizeof(T));
            k.v = pk.zeros(rows * gd.kv_heads * gd.vdim, sizeof(T));
        }
        L->kept.push_back(k);
    }
    return pk.rc;
}

template <typename T> const DecoderOps* hybrid_ops() {
    static const DecoderOps ops{hybrid_alloc_scratch<T>, hybrid_run_layers<T>, true, hybrid_graph_step, hybrid_gemms_per_step, nullptr};
    return &ops;
}

int hybrid_build(b200p_session* s, const b200p_model* m) {
    if (s->dtype != B200P_BF16 && s->dtype != B200P_F32) return B200P_E_DTYPE;
    auto L = std::make_shared<HybridState>();
    L->spec = *std::static_pointer_cast<HybridSpec>(m->spec);
    s->decoder = L;
    s->ops = s->dtype == B200P_F32 ? hybrid_ops<float>() : hybrid_ops<__nv_bfloat16>();
    s->H = L->H = pad16(L->spec.width);
    s->eps = float(L->spec.eps);
    s->embed_scale = float(L->spec.embed_scale);
    for (const HybridLayer& ly : L->spec.layers) {
        L->max_ff = std::max(L->max_ff, pad16(ly.ff)); L->max_main = std::max(L->max_main, ly.main_row()); L->max_ab = std::max(L->max_ab, ly.ab_row());
        L->max_v = std::max(L->max_v, ly.v_row());
    }
    for (const HybridSpec::Pass& p : L->spec.passes) L->looped = L->looped || p.embed_again;
    if (int rc = s->dtype == B200P_F32 ? build_weights<float>(s, m) : build_weights<__nv_bfloat16>(s, m)) return rc;
    s->skinny_max_k = L->H;
    s->skinny_usable = s->dtype != B200P_F32;
    if (cudaError_t e = s->alloc(&s->d_attn_status, 16)) return int(e);
    return int(cudaMemset(s->d_attn_status, 0, 16));
}

const ArchitectureEntry entry("Vofusun", hybrid_configure, hybrid_build);

} // namespace
} // namespace b200p
