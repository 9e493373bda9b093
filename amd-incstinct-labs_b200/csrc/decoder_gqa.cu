// ---------------------------------------------------------------------------
// decoder_gqa.cu -- the Llama-style decoder of the runtime: grouped-query attention with
// rotate-half RoPE, pre-norm, SiLU MLP.
//
// The layers of cdna3::runtime::Session (cdna3-prims/include/cdna3/runtime/
// session.hpp:52-331), its KVCache (kv_cache.hpp:19-52) and the forward kernels of
// forward.hpp:34-262, for a batch of equal-length sequences.
//  * attention reads the token-major projections and the KV cache in place
//    through strided TMA tensor maps, so the four repack_kernel launches per
//    layer and pack_kv are gone (session.hpp:193-207);
//  * RoPE, the optional QKV bias and the scatter into the cache are one kernel;
//    RMSNorm writes the GEMM's 16-bit operand directly; SiLU*up writes the down
//    projection's operand; residual adds are the GEMMs' beta = 1 accumulation;
//  * Q/K/V and gate/up projections are one GEMM each over concatenated weights;
//  * the RoPE table is built once per session, not per step (session.hpp:120-135).
// ---------------------------------------------------------------------------
#include "session.cuh"
#include "decode_mega.cuh"
#include "model.hpp"
#include <cmath>

namespace b200p {
int decode_prepared(const void* q, const void* K, const void* V, void* o, const b200p_decode_args* a,
                    const int* n_dev, int n_add, void* ws, size_t ws_bytes, cudaStream_t st);
int prefill_dispatch_strided(const void* Q, const void* K, const void* V, void* O, const b200p_prefill_cfg* c, int dtype,
                             const b200p_attn_strides* strides, float* debug_s, cudaStream_t st);
namespace {

// forward.hpp:135-148 RoPE (rotate-half) on Q and K in place, rocblas_gemm.hpp:56-63 bias add, and
// forward.hpp:211-224 scatter of K, V into the cache, for token-major qkv [B*T, qd + 2*kvd].
// One thread per (token, head slot, 8 columns d0 .. d0 + 7 < D/2): it owns those and their partners d + D/2, as two
// 16-byte vectors each way.
template <typename T>
__global__ void rope_scatter_kernel(T* __restrict__ qkv, const T* __restrict__ bias, const float* __restrict__ cos_t,
                                    const float* __restrict__ sin_t, T* __restrict__ kcache, T* __restrict__ vcache,
                                    int B, int Tn, int nQH, int nKVH, int D, int pos0, int max_seq,
                                    const int* __restrict__ pos_dev) {
    griddep_launch_dependents();
    if (pos_dev) pos0 = min(*pos_dev, max_seq - Tn);         // device-side position (graph replay), kept inside the cache
    const int half = D / 2, chunks = half / 8;
    const int slots = nQH + 2 * nKVH;                       // q heads, k heads, v heads
    const size_t total = size_t(B) * Tn * slots * chunks;
    const size_t idx = size_t(blockIdx.x) * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const int d0 = int(idx % chunks) * 8;
    const int slot = int((idx / chunks) % slots);
    const size_t tok = idx / (size_t(chunks) * slots);       // b * Tn + s
    const int s = int(tok % Tn), b = int(tok / Tn);
    const int W = slots * D;
    T* row = qkv + tok * W + size_t(slot) * D;
    uint4 va = *reinterpret_cast<const uint4*>(row + d0), vb = *reinterpret_cast<const uint4*>(row + d0 + half);
    T* a = reinterpret_cast<T*>(&va);
    T* h = reinterpret_cast<T*>(&vb);
    const bool rotate = slot < nQH + nKVH;
    if (bias) {                                              // fp16 GEMM output + fp16 bias, rounded (bias_add_f16_kernel)
        const uint4 ba = *reinterpret_cast<const uint4*>(bias + slot * D + d0), bb = *reinterpret_cast<const uint4*>(bias + slot * D + d0 + half);
        const T* pa = reinterpret_cast<const T*>(&ba);
        const T* pb = reinterpret_cast<const T*>(&bb);
        #pragma unroll
        for (int i = 0; i < 8; ++i) { a[i] = from_float<T>(to_float(a[i]) + to_float(pa[i])); h[i] = from_float<T>(to_float(h[i]) + to_float(pb[i])); }
    }
    if (rotate) {
        const int pos = pos0 + s;
        const float4* cp = reinterpret_cast<const float4*>(cos_t + size_t(pos) * half + d0);
        const float4* sp = reinterpret_cast<const float4*>(sin_t + size_t(pos) * half + d0);
        const float4 c0 = cp[0], c1 = cp[1], s0 = sp[0], s1 = sp[1];
        const float cs[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
        const float sn[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
        #pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float x0 = to_float(a[i]), x1 = to_float(h[i]);
            a[i] = from_float<T>(x0 * cs[i] - x1 * sn[i]);   // d < D/2:  t*c + (-t[d+D/2])*s
            h[i] = from_float<T>(x1 * cs[i] + x0 * sn[i]);   // d >= D/2: t*c + ( t[d-D/2])*s
        }
    }
    if (rotate || bias) {
        *reinterpret_cast<uint4*>(row + d0) = va; *reinterpret_cast<uint4*>(row + d0 + half) = vb;
    }
    if (slot >= nQH) {                                       // k or v: into cache[b][kvh][pos][:]
        const bool is_k = slot < nQH + nKVH;
        const int kvh = is_k ? slot - nQH : slot - nQH - nKVH;
        T* dst = (is_k ? kcache : vcache) + ((size_t(b) * nKVH + kvh) * max_seq + pos0 + s) * D;
        *reinterpret_cast<uint4*>(dst + d0) = va; *reinterpret_cast<uint4*>(dst + d0 + half) = vb;
    }
}

template <typename T>
__global__ void concat_rows_kernel(T* __restrict__ dst, const T* __restrict__ a, size_t na, const T* __restrict__ b, size_t nb,
                                   const T* __restrict__ c, size_t nc) {
    const size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x;
    if (i < na) dst[i] = a[i];
    else if (i < na + nb) dst[i] = b[i - na];
    else if (i < na + nb + nc) dst[i] = c[i - na - nb];
}

struct GqaState {
    int qd = 0, kvd = 0, W = 0;
    std::vector<b200p_layer_weights> layers;
    std::vector<void*> Wqkv, Wgu, bqkv;                 // session-owned concatenations
    float *gu = nullptr, *cos_t = nullptr, *sin_t = nullptr;
    void *norm = nullptr, *qkv = nullptr, *attn = nullptr, *act = nullptr;
    void *kcache = nullptr, *vcache = nullptr, *decode_ws = nullptr;
    size_t decode_ws_bytes = 0, layer_cache_elems = 0;
    // the decode loop as one persistent kernel (decode_mega.cuh): per-layer pointer table, split scratch, counters
    MegaLayer* mega_layers = nullptr;
    float* mega_part = nullptr;
    unsigned* mega_words = nullptr;                      // [0] grid barrier, [1] key readers
};
GqaState* gqa(const b200p_session* s) { return static_cast<GqaState*>(s->decoder.get()); }

int gqa_alloc_scratch(b200p_session* s, int M) {
    GqaState* d = gqa(s);
    const auto& c = s->c;
    cudaError_t e;
    if ((e = s->alloc_scratch(&d->norm, size_t(M) * c.hidden * 2))) return int(e);
    if ((e = s->alloc_scratch(&d->qkv, size_t(M) * d->W * 2))) return int(e);
    if ((e = s->alloc_scratch(&d->attn, size_t(M) * d->qd * 2))) return int(e);
    if ((e = s->alloc_scratch(&d->gu, size_t(M) * 2 * c.ffn_dim * 4))) return int(e);
    return int(s->alloc_scratch(&d->act, size_t(M) * c.ffn_dim * 2));
}

// One decoder layer of the decode step (one new token per sequence) on the skinny kernels:
// norm+QKV, RoPE/scatter, attention, O (+= residual), norm+gate/up+SiLU, down (+= residual).
template <typename T>
int decode_layer_skinny(b200p_session* s, int li, int pos0, cudaStream_t st, const int* pos_dev) {
    const GqaState* d = gqa(s);
    const auto& c = s->c;
    const int H = c.hidden, F = c.ffn_dim, D = c.head_dim, B = s->batch;
    const int qd = d->qd, W = d->W;
    const b200p_layer_weights& L = d->layers[li];
    T* kc = static_cast<T*>(d->kcache) + size_t(li) * d->layer_cache_elems;
    T* vc = static_cast<T*>(d->vcache) + size_t(li) * d->layer_cache_elems;
    SkinnyArgs a{};
    a.M = B; a.eps = 1e-6f; a.abort_word = s->d_abort;
    a.W = d->Wqkv[li]; a.X32 = s->hidden; a.norm_w = L.norm_attn; a.out = d->qkv; a.N = W; a.K = H; a.ldo = W;
    if (tuning(KNOB_RUNTIME_ROPE_FUSED, 1) != 0) {
        // 1.-4. attention RMSNorm, Q/K/V projection, bias, RoPE and the K/V scatter into the cache: one kernel
        a.rope.bias = d->bqkv[li]; a.rope.cos_t = d->cos_t; a.rope.sin_t = d->sin_t; a.rope.kcache = kc; a.rope.vcache = vc;
        a.rope.pos_dev = pos_dev; a.rope.pos0 = pos0; a.rope.nQH = c.n_heads; a.rope.nKVH = c.n_kv_heads; a.rope.D = D; a.rope.max_seq = s->max_seq;
        if (int e = launch_skinny<T, PRO_RMSNORM, EPI_ROPE>(a, st)) return e;
    } else {
        // 1.+2. attention RMSNorm fused into the Q/K/V projection; 3.+4. bias, RoPE, K/V into the cache
        if (int e = launch_skinny<T, PRO_RMSNORM, EPI_STORE16>(a, st)) return e;
        const size_t n = size_t(B) * (c.n_heads + 2 * c.n_kv_heads) * (D / 16);
        rope_scatter_kernel<T><<<blocks(n), 256, 0, st>>>(static_cast<T*>(d->qkv), static_cast<const T*>(d->bqkv[li]),
                                                          d->cos_t, d->sin_t, kc, vc, B, 1, c.n_heads, c.n_kv_heads, D, pos0, s->max_seq, pos_dev);
        launched();
    }
    // 5. attention over the cache
    {
        b200p_decode_args da{};
        da.D = D; da.N = pos_dev ? s->max_seq : pos0 + 1; da.nQHeads = c.n_heads; da.nKVHeads = c.n_kv_heads; da.stride_kv = s->max_seq;
        da.batch = B; da.dtype = s->dtype; da.kv_batch_stride = (long long)c.n_kv_heads * s->max_seq * D;
        da.key_offset = 0; da.q_batch_stride = W; da.o_batch_stride = qd;
        // the session's workspace stays prepared (zeroed at creation): no clearing memset per layer
        if (int e = decode_prepared(d->qkv, kc, vc, d->attn, &da, pos_dev, 1, d->decode_ws, d->decode_ws_bytes, st)) return e;
    }
    // 6. O projection accumulated into the residual stream
    a = SkinnyArgs{}; a.M = B; a.eps = 1e-6f; a.abort_word = s->d_abort;
    a.W = L.Wo; a.X16 = d->attn; a.ldx = qd; a.out = s->hidden; a.N = H; a.K = qd; a.ldo = H;
    if (int e = launch_skinny<T, PRO_PLAIN, EPI_ACC32>(a, st)) return e;
    // 7.+8. MLP RMSNorm fused into gate/up, SiLU(gate) * up as the epilogue
    a = SkinnyArgs{}; a.M = B; a.eps = 1e-6f; a.abort_word = s->d_abort;
    a.W = d->Wgu[li]; a.X32 = s->hidden; a.norm_w = L.norm_mlp; a.out = d->act; a.N = F; a.K = H; a.ldo = F;
    if (int e = launch_skinny<T, PRO_RMSNORM, EPI_SILU16>(a, st)) return e;
    //    down projection accumulated into the residual stream
    a = SkinnyArgs{}; a.M = B; a.eps = 1e-6f; a.abort_word = s->d_abort;
    a.W = L.Wdown; a.X16 = d->act; a.ldx = F; a.out = s->hidden; a.N = H; a.K = F; a.ldo = H;
    if (int e = launch_skinny<T, PRO_PLAIN, EPI_ACC32>(a, st)) return e;
    s->gemm_calls += 4;
    return B200P_OK;
}

template <typename T>
int gqa_run_layers(b200p_session* s, int Tn, int pos0, cudaStream_t st, const int* pos_dev) {
    const GqaState* d = gqa(s);
    const auto& c = s->c;
    const int H = c.hidden, F = c.ffn_dim, D = c.head_dim, B = s->batch, M = B * Tn;
    const int qd = d->qd, W = d->W;
    s->final_x = s->hidden;
    if (Tn == 1 && skinny_ok(s, M)) {
        for (int li = 0; li < c.n_layers; ++li)
            if (int e = decode_layer_skinny<T>(s, li, pos0, st, pos_dev)) return e;
        return B200P_OK;
    }
    for (int li = 0; li < c.n_layers; ++li) {
        const b200p_layer_weights& L = d->layers[li];
        T* kc = static_cast<T*>(d->kcache) + size_t(li) * d->layer_cache_elems;
        T* vc = static_cast<T*>(d->vcache) + size_t(li) * d->layer_cache_elems;
        // 1. attention RMSNorm -> 16-bit operand
        rmsnorm_cast_kernel<T><<<blocks(size_t(M) * 32), 256, 0, st>>>(s->hidden, static_cast<const T*>(L.norm_attn), static_cast<T*>(d->norm), M, H, H, 1e-6f, 1, 0);
        launched();
        // 2. Q, K, V projections in one GEMM -> qkv [M, qd + 2 kvd] 16-bit
        if (int e = session_gemm(s, d->norm, d->Wqkv[li], d->qkv, M, W, H, H, W, false, false, st)) return e;
        // 3.+4. bias, RoPE on Q and K, K/V into the cache at [pos0, pos0 + Tn)
        {
            const size_t n = size_t(M) * (c.n_heads + 2 * c.n_kv_heads) * (D / 16);
            rope_scatter_kernel<T><<<blocks(n), 256, 0, st>>>(static_cast<T*>(d->qkv), static_cast<const T*>(d->bqkv[li]),
                                                              d->cos_t, d->sin_t, kc, vc, B, Tn, c.n_heads, c.n_kv_heads, D, pos0, s->max_seq, pos_dev);
            launched();
        }
        // 5. attention over the cache, in place
        if (Tn > 1) {
            if (pos0 != 0) return B200P_E_OP;                 // like the reference, prefill starts from an empty cache
            b200p_prefill_cfg pc{D, Tn, Tn, c.n_heads, c.n_kv_heads, B, 1};
            b200p_attn_strides a{};
            a.q_seq = W; a.q_head = D; a.q_batch = (long long)Tn * W;
            a.k_seq = D; a.k_head = (long long)s->max_seq * D; a.k_batch = (long long)c.n_kv_heads * s->max_seq * D;
            a.v_seq = a.k_seq; a.v_head = a.k_head; a.v_batch = a.k_batch;
            a.o_seq = qd; a.o_head = D; a.o_batch = (long long)Tn * qd;
            if (int e = prefill_dispatch_strided(d->qkv, kc, vc, d->attn, &pc, s->dtype, &a, nullptr, st)) return e;
        } else {
            b200p_decode_args a{};
            a.D = D; a.N = pos0 + 1; a.nQHeads = c.n_heads; a.nKVHeads = c.n_kv_heads; a.stride_kv = s->max_seq;
            a.batch = B; a.dtype = s->dtype; a.kv_batch_stride = (long long)c.n_kv_heads * s->max_seq * D;
            a.key_offset = 0; a.q_batch_stride = W; a.o_batch_stride = qd;
            if (pos_dev) {                                      // key count = *pos_dev + 1, bound = the cache length
                a.N = s->max_seq;
                if (int e = b200p_attn_decode_dyn(d->qkv, kc, vc, d->attn, &a, pos_dev, 1, d->decode_ws, d->decode_ws_bytes, st)) return e;
            } else if (int e = b200p_attn_decode(d->qkv, kc, vc, d->attn, &a, d->decode_ws, d->decode_ws_bytes, st)) return e;
        }
        // 6. O projection, accumulated into the residual stream
        if (int e = session_gemm(s, d->attn, L.Wo, s->hidden, M, H, qd, qd, H, true, true, st)) return e;
        // 7. MLP RMSNorm
        rmsnorm_cast_kernel<T><<<blocks(size_t(M) * 32), 256, 0, st>>>(s->hidden, static_cast<const T*>(L.norm_mlp), static_cast<T*>(d->norm), M, H, H, 1e-6f, 1, 0);
        launched();
        // 8. gate and up in one GEMM with SiLU(gate) * up as its epilogue (or, through the GEMM library: fp32 out and a
        //    separate kernel), down accumulated into the residual stream
        int fused = B200P_E_RANGE;
        if (tuning(KNOB_RUNTIME_GEMM, 1) != 0) {
            fused = gemm_tc(s->dtype, GEMM_EPI_SILU16, d->norm, d->Wgu[li], d->act, M, F, H, H, H, F, st);
            if (fused == B200P_OK) ++s->gemm_calls;
            else if (fused != B200P_E_RANGE && fused != B200P_E_ALIGN) return fused;
        }
        if (fused != B200P_OK) {
            if (int e = session_gemm(s, d->norm, d->Wgu[li], d->gu, M, 2 * F, H, H, 2 * F, true, false, st)) return e;
            silu_mul_cast_kernel<T><<<blocks(size_t(M) * F), 256, 0, st>>>(d->gu, static_cast<T*>(d->act), size_t(M), F);
            launched();
        }
        if (int e = session_gemm(s, d->act, L.Wdown, s->hidden, M, H, F, F, H, true, true, st)) return e;
    }
    return B200P_OK;
}

// ---- the decode loop as one persistent kernel (decode_mega.cuh) ---------------------------------------
struct MegaPlan { const void* kernel = nullptr; int nstages = 0, x_bytes = 0, tab_bytes = 0, stage_bytes = 0; size_t dyn = 0; };

template <typename T>
const void* mega_kernel(int D) {
    return D == 64 ? reinterpret_cast<const void*>(decode_mega_kernel<T, 2>) : D == 128 ? reinterpret_cast<const void*>(decode_mega_kernel<T, 4>) : nullptr;
}

// Whether (and how) this session's decode steps run as the persistent kernel: the projection kernels' domain,
// at most 8 sequences, heads of 64 or 128 columns, a device that launches
// cooperatively, and room for at least two weight stages beside X.
template <typename T>
bool mega_plan(const b200p_session* s, MegaPlan* out) {
    const GqaState* d = gqa(s);
    const auto& c = s->c;
    if (tuning(KNOB_RUNTIME_MEGA, 0) == 0 || tuning(KNOB_RUNTIME_SKINNY, 2) != 2 || !d->mega_layers) return false;
    if (!skinny_ok(s, s->batch) || s->batch > kMegaMaxRows || c.n_kv_heads < 1 || c.n_heads % c.n_kv_heads != 0) return false;
    const int D = c.head_dim;
    MegaPlan pl;
    pl.kernel = mega_kernel<T>(D);
    if (!pl.kernel || device_status_ptr() == nullptr) return false;
    const int B = s->batch, Mp = B <= 1 ? 1 : B <= 2 ? 2 : B <= 4 ? 4 : 8;
    const int maxK = std::max(std::max(c.hidden, c.ffn_dim), d->qd);
    const int slab = std::min(kSkinnySlab, maxK);
    const size_t x_need = size_t(Mp) * (maxK + kSkinnyXPad) * 2;
    const size_t att_need = size_t(kSkinnyWarps) * (2 * D + 2) * sizeof(float);
    pl.x_bytes = int((std::max(x_need, att_need) + 127) / 128 * 128);
    pl.stage_bytes = 16 * (slab * 2 + 16);
    const int budget = 232448 - 8704;                          // shared memory per CTA minus the kernel's static part
    pl.tab_bytes = int((size_t(c.n_layers) * sizeof(MegaLayer) + 127) / 128 * 128);
    pl.nstages = std::min(kSkinnyMaxStages, (budget - pl.x_bytes - pl.tab_bytes) / pl.stage_bytes);
    if (pl.nstages < 2) return false;
    pl.dyn = size_t(pl.x_bytes) + pl.tab_bytes + size_t(pl.nstages) * pl.stage_bytes;
    int dev = 0, coop = 0, per_sm = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&coop, cudaDevAttrCooperativeLaunch, dev) != cudaSuccess || !coop) {
        cudaGetLastError();
        return false;
    }
    if (cudaFuncSetAttribute(pl.kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(pl.dyn)) != cudaSuccess ||
        cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, pl.kernel, kSkinnyStreamThreads, pl.dyn) != cudaSuccess || per_sm < 1) {
        cudaGetLastError();
        return false;
    }
    *out = pl;
    return true;
}

// n_steps decode steps from the device-side state (position, output column) and the ids in ids_in.
template <typename T>
int mega_launch(b200p_session* s, const MegaPlan& pl, const int* ids_in, int n_steps, bool want_argmax, int* tokens, int tokens_stride,
                cudaStream_t st) {
    const GqaState* d = gqa(s);
    const auto& c = s->c;
    if (cudaError_t e = cudaMemsetAsync(d->mega_words, 0, sizeof(unsigned), st)) return int(e);      // the grid barrier's counter
    MegaParams p{};
    p.layers = d->mega_layers; p.n_layers = c.n_layers; p.B = s->batch; p.H = c.hidden; p.F = c.ffn_dim; p.D = c.head_dim;
    p.nQH = c.n_heads; p.nKVH = c.n_kv_heads; p.V = c.vocab_size; p.max_seq = s->max_seq;
    p.embed = s->embed; p.lm_head = s->lm_head; p.final_norm = s->final_norm;
    p.hidden = s->hidden; p.qkv = d->qkv; p.act = d->act; p.logits = s->logits;
    p.kcache = d->kcache; p.vcache = d->vcache; p.layer_cache_elems = d->layer_cache_elems;
    p.cos_t = d->cos_t; p.sin_t = d->sin_t;
    p.part = d->mega_part;
    p.ids_in = ids_in; p.next_ids = s->d_next; p.tokens = tokens; p.tokens_stride = tokens_stride; p.state = s->d_state;
    p.keys = s->d_keys; p.key_ticket = d->mega_words + 1; p.bar = d->mega_words;
    p.status = s->d_abort; p.sticky = device_status_ptr();
    p.n_steps = n_steps; p.want_argmax = want_argmax ? 1 : 0;
    p.nstages = pl.nstages; p.slab_cols = kSkinnySlab; p.x_bytes = pl.x_bytes; p.tab_bytes = pl.tab_bytes; p.stage_bytes = pl.stage_bytes;
    p.ahead = tuning(KNOB_RUNTIME_MEGA_AHEAD, 0);              // measured: 1.03 ms per token without, 1.07 / 1.08 / 1.17 at 2 / 4 / 8 stages
    p.eps = 1e-6f; p.scale_log2 = (1.f / sqrtf(float(c.head_dim))) * 1.4426950408889634f;
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(unsigned(sm_count())); cfg.blockDim = dim3(kSkinnyStreamThreads); cfg.dynamicSmemBytes = pl.dyn; cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeCooperative;
    attr[0].val.cooperative = 1;
    cfg.attrs = attr; cfg.numAttrs = 1;
    void* args[] = {&p};
    const cudaError_t le = cudaLaunchKernelExC(&cfg, pl.kernel, args);
    if (le != cudaSuccess) { cudaGetLastError(); return int(le); }
    g_launches.fetch_add(1, std::memory_order_relaxed);
    ++s->mega_launches;
    s->gemm_calls += (unsigned long long)(n_steps) * (4ull * c.n_layers + 1);
    return B200P_OK;
}

template <typename T>
int gqa_decode_loop(b200p_session* s, const int* ids_in, int n_steps, bool want_argmax, int* tokens, int tokens_stride,
                    cudaStream_t st, bool* handled) {
    MegaPlan pl;
    *handled = mega_plan<T>(s, &pl);
    return *handled ? mega_launch<T>(s, pl, ids_in, n_steps, want_argmax, tokens, tokens_stride, st) : B200P_OK;
}

bool gqa_graph_step(const b200p_session*) { return true; }
int gqa_gemms_per_step(const b200p_session* s) { return 4 * s->c.n_layers; }

template <typename T>
int gqa_build(b200p_session* s) {
    GqaState* d = gqa(s);
    const auto& c = s->c;
    const int H = c.hidden, F = c.ffn_dim, D = c.head_dim;
    cudaError_t e;
    for (int li = 0; li < c.n_layers; ++li) {
        const b200p_layer_weights& L = d->layers[li];
        T *wqkv = nullptr, *wgu = nullptr, *b = nullptr;
        const size_t nq = size_t(d->qd) * H, nk = size_t(d->kvd) * H, nf = size_t(F) * H;
        if ((e = s->alloc(&wqkv, (nq + 2 * nk) * 2))) return int(e);
        if ((e = s->alloc(&wgu, 2 * nf * 2))) return int(e);
        concat_rows_kernel<T><<<blocks(nq + 2 * nk), 256>>>(wqkv, (const T*)L.Wq, nq, (const T*)L.Wk, nk, (const T*)L.Wv, nk);
        concat_rows_kernel<T><<<blocks(2 * nf), 256>>>(wgu, (const T*)L.Wgate, nf, (const T*)L.Wup, nf, (const T*)nullptr, 0);
        launched(2);
        if (L.bq && L.bk && L.bv) {
            if ((e = s->alloc(&b, size_t(d->W) * 2))) return int(e);
            concat_rows_kernel<T><<<blocks(d->W), 256>>>(b, (const T*)L.bq, d->qd, (const T*)L.bk, d->kvd, (const T*)L.bv, d->kvd);
            launched();
        }
        d->Wqkv.push_back(wqkv); d->Wgu.push_back(wgu); d->bqkv.push_back(b);
    }
    // RoPE table, session.hpp:120-135: freq = 1 / theta^(2d/D), angle = pos * freq
    std::vector<float> cosv(size_t(s->max_seq) * D / 2), sinv(cosv.size());
    for (int pos = 0; pos < s->max_seq; ++pos)
        for (int d = 0; d < D / 2; ++d) {
            const float freq = 1.f / powf(c.rope_theta, (2.f * d) / D);
            const float ang = pos * freq;
            cosv[size_t(pos) * (D / 2) + d] = cosf(ang);
            sinv[size_t(pos) * (D / 2) + d] = sinf(ang);
        }
    if ((e = s->alloc(&d->cos_t, cosv.size() * 4))) return int(e);
    if ((e = s->alloc(&d->sin_t, sinv.size() * 4))) return int(e);
    if ((e = cudaMemcpy(d->cos_t, cosv.data(), cosv.size() * 4, cudaMemcpyHostToDevice))) return int(e);
    if ((e = cudaMemcpy(d->sin_t, sinv.data(), sinv.size() * 4, cudaMemcpyHostToDevice))) return int(e);
    // KV cache [L][B][kvh][max_seq][D], zero-filled like kv_cache.hpp:34-37
    d->layer_cache_elems = size_t(s->batch) * c.n_kv_heads * s->max_seq * D;
    const size_t cache_bytes = size_t(c.n_layers) * d->layer_cache_elems * 2;
    if ((e = s->alloc(&d->kcache, cache_bytes))) return int(e);
    if ((e = s->alloc(&d->vcache, cache_bytes))) return int(e);
    if ((e = cudaMemset(d->kcache, 0, cache_bytes))) return int(e);
    if ((e = cudaMemset(d->vcache, 0, cache_bytes))) return int(e);
    // caller-owned weights the skinny kernels stream: misaligned views take the library GEMMs instead
    s->skinny_max_k = std::max(c.ffn_dim, c.hidden);
    s->skinny_usable = c.hidden % 16 == 0 && c.ffn_dim % 16 == 0 && d->qd % 16 == 0 && aligned(s->lm_head, 16) && aligned(s->final_norm, 8);
    for (const auto& L : d->layers)
        s->skinny_usable = s->skinny_usable && aligned(L.Wo, 16) && aligned(L.Wdown, 16) && aligned(L.norm_attn, 8) && aligned(L.norm_mlp, 8);
    // the persistent decode kernel's tables and scratch (decode_mega.cuh), when the shape is in its domain
    if (s->batch <= kMegaMaxRows && c.n_heads / c.n_kv_heads <= kMegaMaxGroup) {
        std::vector<MegaLayer> ml(c.n_layers);
        for (int li = 0; li < c.n_layers; ++li) {
            const b200p_layer_weights& L = d->layers[li];
            ml[li] = MegaLayer{d->Wqkv[li], d->bqkv[li], L.Wo, d->Wgu[li], L.Wdown, L.norm_attn, L.norm_mlp};
        }
        const size_t units = size_t(s->batch) * c.n_heads;
        if ((e = s->alloc(&d->mega_layers, ml.size() * sizeof(MegaLayer)))) return int(e);
        if ((e = cudaMemcpy(d->mega_layers, ml.data(), ml.size() * sizeof(MegaLayer), cudaMemcpyHostToDevice))) return int(e);
        if ((e = s->alloc(&d->mega_part, units * kMegaMaxSplits * kMegaPartPad(D) * sizeof(float)))) return int(e);
        if ((e = s->alloc(&d->mega_words, 2 * sizeof(unsigned)))) return int(e);
        if ((e = cudaMemset(d->mega_words, 0, 2 * sizeof(unsigned)))) return int(e);
    }
    // decode scratch for the longest cache
    b200p_decode_args a{};
    a.D = D; a.N = s->max_seq; a.nQHeads = c.n_heads; a.nKVHeads = c.n_kv_heads; a.stride_kv = s->max_seq; a.batch = s->batch; a.dtype = s->dtype;
    size_t need = 0;
    for (int n = 1; n <= s->max_seq; n = n < 128 ? 128 : n * 2) {       // the split plan depends on N: take the largest need
        a.N = n < s->max_seq ? n : s->max_seq;
        const size_t b = b200p_attn_decode_workspace_bytes(&a);
        need = b > need ? b : need;
        if (a.N == s->max_seq) break;
    }
    d->decode_ws_bytes = need * 2;
    if ((e = s->alloc(&d->decode_ws, d->decode_ws_bytes))) return int(e);
    if ((e = cudaMemset(d->decode_ws, 0, d->decode_ws_bytes))) return int(e);
    s->d_attn_status = static_cast<int*>(d->decode_ws);       // the status word at the head of the decode workspace
    return B200P_OK;
}

template <typename T> const DecoderOps* gqa_ops() {
    static const DecoderOps ops{gqa_alloc_scratch, gqa_run_layers<T>, false, gqa_graph_step, gqa_gemms_per_step, gqa_decode_loop<T>};
    return &ops;
}

} // namespace
} // namespace b200p

using namespace b200p;

extern "C" b200p_session* b200p_session_create(const b200p_model_weights* w, int max_seq, int batch, int* status) {
    int dummy; if (!status) status = &dummy;
    *status = B200P_OK;
    if (!w || !w->layers || !w->embed_tokens || !w->lm_head || !w->final_norm) { *status = B200P_E_NULL; return nullptr; }
    if (w->dtype != B200P_F16 && w->dtype != B200P_BF16) { *status = B200P_E_DTYPE; return nullptr; }
    const auto& c = w->cfg;
    if ((c.head_dim != 64 && c.head_dim != 128) || c.n_heads <= 0 || c.n_kv_heads <= 0 || c.n_heads % c.n_kv_heads != 0 ||
        c.hidden % 8 != 0 || c.ffn_dim % 8 != 0) { *status = B200P_E_DIM; return nullptr; }
    if (max_seq <= 0 || batch <= 0 || c.n_layers <= 0 || c.vocab_size <= 0) { *status = B200P_E_LENGTH; return nullptr; }
    if (sm_count() <= 0) { *status = B200P_E_NO_DEVICE; return nullptr; }
    b200p_session* s = new b200p_session();
    s->c = c; s->dtype = w->dtype; s->max_seq = max_seq; s->batch = batch;
    s->H = c.hidden;
    auto d = std::make_shared<GqaState>();
    s->decoder = d;
    s->ops = w->dtype == B200P_F16 ? gqa_ops<__half>() : gqa_ops<__nv_bfloat16>();
    d->qd = c.n_heads * c.head_dim; d->kvd = c.n_kv_heads * c.head_dim; d->W = d->qd + 2 * d->kvd;
    s->embed = w->embed_tokens; s->lm_head = w->lm_head; s->final_norm = w->final_norm;
    d->layers.assign(w->layers, w->layers + c.n_layers);
    for (const auto& L : d->layers)
        if (!L.Wq || !L.Wk || !L.Wv || !L.Wo || !L.Wgate || !L.Wup || !L.Wdown || !L.norm_attn || !L.norm_mlp) {
            *status = B200P_E_NULL; delete s; return nullptr;
        }
    int rc = session_common_init(s);
    if (!rc) rc = w->dtype == B200P_F16 ? gqa_build<__half>(s) : gqa_build<__nv_bfloat16>(s);
    if (!rc) rc = int(cudaDeviceSynchronize());
    if (rc) { *status = rc; b200p_session_destroy(s); return nullptr; }
    return s;
}

namespace { const bool registered = (llama_session_create() = b200p_session_create, true); }
