// ---------------------------------------------------------------------------
// session.cuh -- what the parts of the LLM runtime share: the session object, the
// interface between the session (runtime.cu: entry points, scratch, embedding,
// logits, sampling, the greedy loop and its step graph) and its decoder
// (decoder_gqa.cu: Llama-style; decoder_latent.cu: latent attention; decoder_hybrid.cu:
// gated delta rule and masked attention), and the row kernels that they share.
// ---------------------------------------------------------------------------
#pragma once
#include "common.cuh"
#include "attn_common.cuh"
#include "mma_sync.cuh"
#include "skinny_gemm.cuh"
#include "vec_quads.cuh"
#include "gemm_tc.cuh"
#include "wave_primitives/wave64.cuh"
#include "b200p_runtime.h"
#include <cublas_v2.h>
#include <memory>
#include <vector>

struct b200p_session;

namespace b200p {

// A decoder: what happens between the embedding and the final norm, for a batch of equal-length sequences.
struct DecoderOps {
    // Activation buffers for M rows (tokens of all sequences); called when M exceeds every earlier call's.
    // The session has synchronised, dropped its step graph and released s->scratch before.
    int (*alloc_scratch)(b200p_session* s, int M);
    // The Tn tokens of every sequence whose embeddings are in s->hidden, at positions pos0 .. pos0 + Tn - 1 (decode
    // steps: *pos_dev, read on the device), through all layers and into the cache.  Leaves the residual stream in
    // s->final_x.  pos0 = 0 starts new sequences: whatever the cache or a recurrent state holds does not count.
    int (*run_layers)(b200p_session* s, int Tn, int pos0, cudaStream_t st, const int* pos_dev);
    bool portions;                             // run_layers takes Tn > 1 at pos0 > 0
    bool (*graph_step)(const b200p_session* s);   // a decode step reads its position on the device only: it can be captured
    int (*gemms_per_step)(const b200p_session* s);
    // Optional: n_steps decode steps in one launch.  *handled = false: not available for this session, nothing done.
    int (*decode_loop)(b200p_session* s, const int* ids_in, int n_steps, bool want_argmax, int* tokens, int tokens_stride,
                       cudaStream_t st, bool* handled);
};

inline unsigned blocks(size_t n, int tpb = 256) { return unsigned((n + tpb - 1) / tpb); }

// forward.hpp:34-56 RMSNorm (y = x * rsqrt(mean(x^2) + eps) * w), writing the GEMM's operand.
// Output row r is the norm of source row r * src_row_stride + src_row_offset (stride > 1: the last token of each
// sequence), or of row (r / n_want) * src_row_stride + want[r % n_want] when `want` is given.  One warp per row: up to
// 16 float4 loads per lane kept in registers between the sum of squares and the scaling (longer rows are read twice,
// the second time from cache), vector stores.  H, the row length, must be a multiple of 4; n is the number of columns
// the mean is over (columns past it are zero padding).
template <typename T>
__global__ void __launch_bounds__(256)
rmsnorm_cast_kernel(const float* __restrict__ X, const T* __restrict__ W, T* __restrict__ Y,
                    int rows, int H, int n, float eps, int src_row_stride, int src_row_offset,
                    const int* __restrict__ want = nullptr, int n_want = 1) {
    const int r = blockIdx.x * (blockDim.x / 32) + threadIdx.x / 32, lane = threadIdx.x % 32;
    if (r >= rows) return;
    const size_t src = want ? size_t(r / n_want) * src_row_stride + want[r % n_want] : size_t(r) * src_row_stride + src_row_offset;
    const float4* x = reinterpret_cast<const float4*>(X + src * H);
    T* y = Y + size_t(r) * H;
    const int quads = H / 4;
    constexpr int CACHE = 16;                                 // quads per lane held in registers: rows up to 2048 floats
    float4 c[CACHE];
    float ss = 0.f;
    #pragma unroll
    for (int i = 0; i < CACHE; ++i) {
        const int q = lane + 32 * i;
        if (q < quads) { c[i] = x[q]; ss += c[i].x * c[i].x + c[i].y * c[i].y + c[i].z * c[i].z + c[i].w * c[i].w; }
    }
    for (int q = lane + 32 * CACHE; q < quads; q += 32) { const float4 v = x[q]; ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
    const float inv = rsqrtf(wave::dpp::reduce_sum(ss) / n + eps);
    const bool w_vec = (reinterpret_cast<uintptr_t>(W) & (4 * sizeof(T) - 1)) == 0;      // caller-owned weights may be any aligned view
    auto put = [&](int q, const float4& v) {
        const float4 w = w_vec ? load4<T>(W + 4 * q)
                               : make_float4(to_float(W[4 * q]), to_float(W[4 * q + 1]), to_float(W[4 * q + 2]), to_float(W[4 * q + 3]));
        store4<T>(y + 4 * q, make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w));
    };
    #pragma unroll
    for (int i = 0; i < CACHE; ++i) { const int q = lane + 32 * i; if (q < quads) put(q, c[i]); }
    for (int q = lane + 32 * CACHE; q < quads; q += 32) put(q, x[q]);
}

// forward.hpp:154-160: silu(gate) * up in fp32, written as the down projection's 16-bit operand.
// gu is [M, 2F]: gate in the first F columns, up in the last F.
template <typename T>
__global__ void silu_mul_cast_kernel(const float* __restrict__ gu, T* __restrict__ act, size_t M, int F) {
    const size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x;
    if (i >= M * F) return;
    const size_t m = i / F; const int f = int(i % F);
    const float g = gu[m * 2 * F + f], u = gu[m * 2 * F + F + f];
    act[i] = from_float<T>((g / (1.f + expf(-g))) * u);
}

} // namespace b200p

struct b200p_session {
    b200p_model_config c{};
    const b200p::DecoderOps* ops = nullptr;
    std::shared_ptr<void> decoder;                       // the decoder's own state
    int dtype = B200P_BF16, max_seq = 0, batch = 0, kv_len = 0, cap_tokens = 0, cap_new = 0, cap_want = 0;
    int H = 0;                                           // row length of the residual stream: hidden, or hidden padded with zero columns
    float eps = 1e-6f;
    float embed_scale = 1.f;
    const void *embed = nullptr, *lm_head = nullptr, *final_norm = nullptr;     // rows of H elements
    cublasHandle_t blas = nullptr;
    void* blas_ws = nullptr;
    static constexpr size_t kBlasWsBytes = size_t(64) << 20;
    float *hidden = nullptr, *logits = nullptr;
    float* embedded = nullptr;                           // a decoder that reads the embeddings again: a second copy of them (its scratch), or null
    const float* final_x = nullptr;                      // the residual stream after the last layer [batch * Tn][H]
    void* last_norm = nullptr;
    float* want_logits = nullptr; void* want_norm = nullptr; int* d_want = nullptr;     // logits at asked places, cap_want rows
    int *d_ids = nullptr, *d_next = nullptr, *d_tokens = nullptr, *d_state = nullptr;
    int* d_abort = nullptr;                              // abort word of the session's streaming kernels (cleared per call, read after it)
    int* d_attn_status = nullptr;                        // status word of the decoder's attention workspace
    bool skinny_usable = true;                           // shapes and alignments are in the skinny kernels' domain ...
    int skinny_max_k = 0;                                // ... with this longest row of X
    unsigned long long* d_keys = nullptr;                // argmax merge keys [batch], zero between launches
    unsigned int* d_tickets = nullptr;                   // argmax arrival counters [batch]
    // one decode step (embed -> layers -> logits -> argmax -> advance) as an executable graph
    cudaStream_t capture_stream = nullptr;
    cudaGraphExec_t step_graph = nullptr;
    const void* graph_hidden = nullptr; const int* graph_tokens = nullptr; int graph_max_new = 0; unsigned graph_epoch = 0;
    unsigned long long graph_replays = 0, graph_kernels = 0;   // kernels of this library inside one replay
    unsigned long long gemm_calls = 0, blas_calls = 0;      // all projections / those that went to the GEMM library
    unsigned long long mega_launches = 0;
    std::vector<void*> owned, scratch;                   // for the session's life / for the current cap_tokens

    template <typename P> cudaError_t alloc(P** p, size_t bytes) { return alloc_in(owned, p, bytes); }
    template <typename P> cudaError_t alloc_scratch(P** p, size_t bytes) { return alloc_in(scratch, p, bytes); }
    template <typename P> static cudaError_t alloc_in(std::vector<void*>& list, P** p, size_t bytes) {
        cudaError_t e = cudaMalloc(reinterpret_cast<void**>(p), bytes ? bytes : 16);
        if (e == cudaSuccess) list.push_back(*p);
        return e;
    }
};

namespace b200p {

// C[M,N] (row-major) = A[M,K] . W[N,K]^T (+ C if accumulate); A, W of the session's type, fp32 accumulation.  16-bit: this
// library's tensor-core GEMM, the GEMM library outside its domain; fp32: the GEMM library in true fp32.
int session_gemm(b200p_session* s, const void* A, const void* Wt, void* Cm, int M, int N, int K, int lda, int ldc, bool c_is_f32,
                 bool accumulate, cudaStream_t st);

// Whether M rows run on the skinny kernels (few rows: a stream over the weights with the norm / activation / residual
// work fused in) instead of GEMMs.
inline bool skinny_ok(const b200p_session* s, int M) {
    return tuning(KNOB_RUNTIME_SKINNY, 2) != 0 && s->skinny_usable && M <= kSkinnyMaxM &&
           size_t(M <= 1 ? 1 : M <= 2 ? 2 : M <= 4 ? 4 : M <= 8 ? 8 : 16) * size_t(s->skinny_max_k + kSkinnyXPad) * 2 <= 190 * 1024;
}

// Creates the parts that every session has; s->c, dtype, max_seq, batch, H, eps, ops and the three top tensors are set.
int session_common_init(b200p_session* s);

} // namespace b200p
