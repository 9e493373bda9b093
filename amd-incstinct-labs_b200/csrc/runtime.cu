// ---------------------------------------------------------------------------
// runtime.cu -- the small LLM runtime around the attention kernels: the session.
//
// Stands in for cdna3::runtime::Session (cdna3-prims/include/cdna3/runtime/
// session.hpp:52-331) and the rocBLAS wrappers of rocblas_gemm.hpp:112-209, for
// a batch of equal-length sequences.  Same arithmetic contract as the
// reference: hidden state fp32, weights and GEMM operands 16-bit with fp32
// accumulation, greedy argmax over 16-bit logits.  (A session of a decoder that
// runs in fp32 has fp32 operands and logits instead.)
//
// The layers are a decoder's (session.cuh: DecoderOps); here is what they share:
// scratch, embedding, final norm and logits, sampling, portions of prompts, the
// greedy loop and its step graph.
//  * GEMMs are this library's tensor-core kernel (gemm_tc.cu) or, outside its
//    domain, library calls (cuBLAS), as they are rocBLAS calls in the reference;
//  * the greedy loop keeps the next-token ids on the device: no per-token
//    device-to-host copy (session.hpp:329), one copy at the end.
// ---------------------------------------------------------------------------
#include "session.cuh"
#include "model.hpp"
#include "status_rc.hpp"
#include <algorithm>
#include <type_traits>

namespace b200p {
namespace {

// ---- kernels ------------------------------------------------------------------------------
// forward.hpp:174-183: out[t, :] = float(embed[ids[t], :]), times a scale, and once more to `copy` if it is given
template <typename T>
__global__ void embed_gather_kernel(const T* __restrict__ embed, const int* __restrict__ ids, float* __restrict__ out, float* __restrict__ copy, float scale, int M, int H) {
    griddep_launch_dependents();
    const int t = blockIdx.x;
    if (t >= M) return;
    const T* src = embed + size_t(ids[t]) * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = to_float(src[i]) * scale;
        out[size_t(t) * H + i] = v;
        if (copy) copy[size_t(t) * H + i] = v;
    }
}

// forward.hpp:244-262 argmax over a [V] row of 16-bit logits; ties go to the lowest index.
// The row is spread over gridDim.y blocks: each folds its slice into a 64-bit key
// (order-preserving value bits, then the complemented index) and merges it into keys[row] with
// atomicMax; the last block of a row to arrive (ticket counter) writes the id for the next
// step and the output token, and clears key and counter for the next launch.
template <typename T>
__global__ void argmax_kernel(const float* __restrict__ logits, int V, int* __restrict__ next_ids,
                              int* __restrict__ tokens, int tokens_stride, int step, const int* __restrict__ step_dev,
                              unsigned long long* __restrict__ keys, unsigned int* __restrict__ tickets) {
    griddep_launch_dependents();
    if (step_dev) step = min(*step_dev, tokens_stride - 1);
    __shared__ unsigned long long red[32];
    const int rowi = blockIdx.x;
    const float* row = logits + size_t(rowi) * V;
    const int per = (V + gridDim.y - 1) / gridDim.y;
    const int i0 = blockIdx.y * per, i1 = min(i0 + per, V);
    unsigned long long best = 0;
    for (int i = i0 + threadIdx.x; i < i1; i += blockDim.x) {
        const float v = to_float(from_float<T>(row[i]));                 // the reference's logits are 16-bit
        unsigned u = __float_as_uint(v);
        u = (u & 0x80000000u) ? ~u : (u | 0x80000000u);                  // order-preserving key
        const unsigned long long key = (unsigned long long)u << 32 | (0xffffffffu - unsigned(i));
        best = key > best ? key : best;
    }
    best = wave::dpp::reduce_max(best);                                  // 64-bit butterfly over the warp
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, nw = blockDim.x / 32;
    if (lane == 0) red[warp] = best;
    __syncthreads();
    if (warp == 0) {
        unsigned long long t = lane < nw ? red[lane] : 0ull;
        t = wave::dpp::reduce_max(t);
        if (lane == 0) {
            atomicMax(&keys[rowi], t);
            __threadfence();
            if (atomicAdd(&tickets[rowi], 1u) == gridDim.y - 1) {        // every slice of the row is in
                __threadfence();
                const unsigned long long k = atomicExch(&keys[rowi], 0ull);
                tickets[rowi] = 0u;
                const int id = int(0xffffffffu - unsigned(k & 0xffffffffu));
                next_ids[rowi] = id;
                if (tokens) tokens[size_t(rowi) * tokens_stride + step] = id;
            }
        }
    }
}

// Device-side step state of the greedy loop: state[0] = position of the token being
// decoded (= keys already in the cache), state[1] = column of the output it produces.
__global__ void set_state_kernel(int* state, int pos, int step) { state[0] = pos; state[1] = step; }
__global__ void advance_state_kernel(int* state) { state[0] += 1; state[1] += 1; }


// f(tag) with a value of the session's element type
template <typename F> int with_type(int dtype, F&& f) {
    return dtype == B200P_F16 ? f(__half{}) : dtype == B200P_BF16 ? f(__nv_bfloat16{}) : f(float{});
}

cudaDataType cuda_type(int dtype) { return dtype == B200P_F16 ? CUDA_R_16F : dtype == B200P_BF16 ? CUDA_R_16BF : CUDA_R_32F; }

} // namespace

// (rocblas_gemm.hpp:112-209: transpose/none with the operands swapped.)
int session_gemm(b200p_session* s, const void* A, const void* Wt, void* Cm, int M, int N, int K, int lda, int ldc, bool c_is_f32,
                 bool accumulate, cudaStream_t st) {
    if (s->dtype != B200P_F32 && tuning(KNOB_RUNTIME_GEMM, 1) != 0 && !(accumulate && !c_is_f32)) {
        // this library's tensor-core GEMM; shapes or pointers outside its domain take the library call below
        const int epi = !c_is_f32 ? GEMM_EPI_STORE16 : accumulate ? GEMM_EPI_ACC32 : GEMM_EPI_STORE32;
        const int rc = gemm_tc(s->dtype, epi, A, Wt, Cm, M, N, K, lda, K, ldc, st);
        if (rc == B200P_OK) { ++s->gemm_calls; return rc; }
        if (rc != B200P_E_RANGE && rc != B200P_E_ALIGN) return rc;
    }
    ++s->blas_calls;
    const float alpha = 1.f, beta = accumulate ? 1.f : 0.f;
    cublasSetStream(s->blas, st);
    cublasSetWorkspace(s->blas, s->blas_ws, b200p_session::kBlasWsBytes);   // SetStream resets it; a fixed one is capturable
    const cudaDataType t = cuda_type(s->dtype);
    // fp32 operands: the pedantic mode never takes a reduced-precision (TF32) path
    const cublasComputeType_t ct = s->dtype == B200P_F32 ? CUBLAS_COMPUTE_32F_PEDANTIC : CUBLAS_COMPUTE_32F;
    const cublasStatus_t r = cublasGemmEx(s->blas, CUBLAS_OP_T, CUBLAS_OP_N, N, M, K, &alpha, Wt, t, K, A, t, lda, &beta,
                                          Cm, c_is_f32 ? CUDA_R_32F : t, ldc, ct, CUBLAS_GEMM_DEFAULT);
    ++s->gemm_calls;
    return r == CUBLAS_STATUS_SUCCESS ? B200P_OK : int(cudaErrorUnknown);
}

int session_common_init(b200p_session* s) {
    const auto& c = s->c;
    const size_t B = size_t(s->batch), esz = s->dtype == B200P_F32 ? 4 : 2;
    cudaError_t e;
    if ((e = s->alloc(&s->logits, B * c.vocab_size * 4))) return int(e);
    if ((e = s->alloc(&s->last_norm, B * s->H * esz))) return int(e);
    if ((e = s->alloc(&s->d_next, B * sizeof(int)))) return int(e);
    if ((e = s->alloc(&s->d_state, 2 * sizeof(int)))) return int(e);
    if ((e = s->alloc(&s->d_abort, sizeof(int)))) return int(e);
    if ((e = cudaMemset(s->d_abort, 0, sizeof(int)))) return int(e);
    if ((e = s->alloc(&s->d_keys, B * sizeof(unsigned long long)))) return int(e);
    if ((e = s->alloc(&s->d_tickets, B * sizeof(unsigned int)))) return int(e);
    if ((e = cudaMemset(s->d_keys, 0, B * sizeof(unsigned long long)))) return int(e);
    if ((e = cudaMemset(s->d_tickets, 0, B * sizeof(unsigned int)))) return int(e);
    if ((e = s->alloc(&s->blas_ws, b200p_session::kBlasWsBytes))) return int(e);
    return cublasCreate(&s->blas) == CUBLAS_STATUS_SUCCESS ? B200P_OK : int(cudaErrorUnknown);
}

namespace {

void drop_step_graph(b200p_session* s) {
    if (s->step_graph) cudaGraphExecDestroy(s->step_graph);
    s->step_graph = nullptr;
}

// Scratch for Tn tokens per sequence: grown, never shrunk; the superseded buffers are released once the device is idle.
int ensure_scratch(b200p_session* s, int Tn, int max_new) {
    const int M = s->batch * Tn;
    if (M > s->cap_tokens) {
        cudaError_t e = cudaSuccess;
        if ((e = cudaDeviceSynchronize())) return int(e);
        for (void* q : s->scratch) cudaFree(q);
        s->scratch.clear();
        s->cap_tokens = 0;
        drop_step_graph(s);                                     // a captured step names the old buffers
        if ((e = s->alloc_scratch(&s->hidden, size_t(M) * s->H * 4))) return int(e);
        if ((e = s->alloc_scratch(&s->d_ids, size_t(M) * sizeof(int)))) return int(e);
        if (int rc = s->ops->alloc_scratch(s, M)) return rc;
        s->cap_tokens = M;
    }
    if (max_new > s->cap_new) {
        if (cudaError_t e = s->alloc(&s->d_tokens, size_t(s->batch) * max_new * sizeof(int))) return int(e);
        s->cap_new = max_new;
    }
    return B200P_OK;
}

// Final norm of rows of s->final_x (row r of the result is source row r * stride + offset, or the wanted rows) into dst.
int final_norm_rows(b200p_session* s, void* dst, int rows, int stride, int offset, const int* want, int n_want, cudaStream_t st) {
    return with_type(s->dtype, [&](auto tag) -> int {
        using T = decltype(tag);
        rmsnorm_cast_kernel<T><<<blocks(size_t(rows) * 32), 256, 0, st>>>(s->final_x, static_cast<const T*>(s->final_norm), static_cast<T*>(dst),
                                                                          rows, s->H, s->c.hidden, s->eps, stride, offset, want, n_want);
        return launched();
    });
}

// lm_head over `rows` normalised rows -> fp32 logits [rows, V].  Few rows are the streaming kernel's case, not a
// tensor-core tile's.
int head_rows(b200p_session* s, const void* norm, float* out, int rows, bool few, cudaStream_t st) {
    const auto& c = s->c;
    if (s->dtype == B200P_F32 || !few) return session_gemm(s, norm, s->lm_head, out, rows, c.vocab_size, s->H, s->H, c.vocab_size, true, false, st);
    return with_type(s->dtype, [&](auto tag) -> int {
        using T = decltype(tag);
        if constexpr (std::is_same_v<T, float>) return B200P_E_DTYPE;
        else {
            SkinnyArgs a{};
            a.M = rows; a.eps = s->eps; a.abort_word = s->d_abort;
            a.W = s->lm_head; a.X16 = norm; a.ldx = s->H; a.out = out; a.N = c.vocab_size; a.K = s->H; a.ldo = c.vocab_size;
            ++s->gemm_calls;
            return launch_skinny<T, PRO_PLAIN, EPI_STORE32>(a, st);
        }
    });
}

// final norm of the LAST token of every sequence + lm_head -> fp32 logits [B, V], after a prefill
int last_logits_prefill(b200p_session* s, int Tn, cudaStream_t st) {
    if (int e = final_norm_rows(s, s->last_norm, s->batch, Tn, Tn - 1, nullptr, 1, st)) return e;
    return head_rows(s, s->last_norm, s->logits, s->batch, skinny_ok(s, s->batch) && tuning(KNOB_RUNTIME_GEMM, 1) != 0, st);
}

// The same for the decode step (one token per sequence): final norm fused into lm_head.
int last_logits_step(b200p_session* s, cudaStream_t st) {
    const auto& c = s->c;
    if (!skinny_ok(s, s->batch)) {
        if (int e = final_norm_rows(s, s->last_norm, s->batch, 1, 0, nullptr, 1, st)) return e;
        return head_rows(s, s->last_norm, s->logits, s->batch, false, st);
    }
    return with_type(s->dtype, [&](auto tag) -> int {
        using T = decltype(tag);
        if constexpr (std::is_same_v<T, float>) return B200P_E_DTYPE;
        else {
            SkinnyArgs a{};
            a.M = s->batch; a.eps = s->eps; a.abort_word = s->d_abort; a.norm_n = c.hidden;
            a.W = s->lm_head; a.X32 = s->final_x; a.norm_w = s->final_norm; a.out = s->logits; a.N = c.vocab_size; a.K = s->H; a.ldo = c.vocab_size;
            ++s->gemm_calls;
            return launch_skinny<T, PRO_RMSNORM, EPI_STORE32>(a, st);
        }
    });
}

int embed(b200p_session* s, const int* ids, int M, cudaStream_t st) {
    return with_type(s->dtype, [&](auto tag) -> int {
        using T = decltype(tag);
        embed_gather_kernel<T><<<M, 256, 0, st>>>(static_cast<const T*>(s->embed), ids, s->hidden, s->embedded, s->embed_scale, M, s->H);
        return launched();
    });
}

// Greedy sampling of every sequence's logits into d_next and column `step` of the token table (*step_dev when given).
// argmax: rows x slices of ~2048 logits
int sample(b200p_session* s, int max_new, int step, const int* step_dev, cudaStream_t st) {
    const int V = s->c.vocab_size;
    return with_type(s->dtype, [&](auto tag) -> int {
        using T = decltype(tag);
        argmax_kernel<T><<<dim3(unsigned(s->batch), unsigned((V + 2047) / 2048)), 256, 0, st>>>(
            s->logits, V, s->d_next, s->d_tokens, max_new, step, step_dev, s->d_keys, s->d_tickets);
        return launched();
    });
}

// One greedy decode step with every per-step quantity read on the device: embed the ids the
// previous argmax left in d_next, run the layers at position state[0], argmax into column
// state[1] of the token table, advance the state.  Launch parameters never change, so the
// step can be captured once and replayed.
int decode_step_device_state(b200p_session* s, int max_new, cudaStream_t st) {
    if (int e = embed(s, s->d_next, s->batch, st)) return e;
    if (int e = s->ops->run_layers(s, 1, 0, st, s->d_state)) return e;
    if (int e = last_logits_step(s, st)) return e;
    if (int e = sample(s, max_new, 0, s->d_state + 1, st)) return e;
    advance_state_kernel<<<1, 1, 0, st>>>(s->d_state);
    return launched();
}

// Capture the decode step on the session's own stream (the caller's may be the legacy default
// stream, which cannot be captured) and instantiate it.  The graph bakes in the scratch
// pointers and the token table's row length, so it is rebuilt when those change.  Called only
// after the same step has run once eagerly (modules loaded, attributes set).
int build_step_graph(b200p_session* s, int max_new) {
    drop_step_graph(s);
    if (!s->capture_stream && cudaStreamCreateWithFlags(&s->capture_stream, cudaStreamNonBlocking) != cudaSuccess) {
        cudaGetLastError();
        return B200P_E_NO_DEVICE;
    }
    if (cudaError_t e = cudaStreamBeginCapture(s->capture_stream, cudaStreamCaptureModeThreadLocal)) { cudaGetLastError(); return int(e); }
    const unsigned long long gemms = s->gemm_calls, launches = g_launches.load();
    const int rc = decode_step_device_state(s, max_new, s->capture_stream);
    s->gemm_calls = gemms;                                   // recording is not running: take the counts back
    s->graph_kernels = g_launches.load() - launches;
    g_launches.fetch_sub(s->graph_kernels);
    cudaGraph_t graph = nullptr;
    const cudaError_t ce = cudaStreamEndCapture(s->capture_stream, &graph);
    if (rc || ce != cudaSuccess || !graph) {
        if (graph) cudaGraphDestroy(graph);
        cudaGetLastError();
        return rc ? rc : int(ce ? ce : cudaErrorUnknown);
    }
    const cudaError_t ie = cudaGraphInstantiate(&s->step_graph, graph, 0);
    cudaGraphDestroy(graph);
    if (ie != cudaSuccess) { s->step_graph = nullptr; cudaGetLastError(); return int(ie); }
    s->graph_hidden = s->hidden; s->graph_tokens = s->d_tokens; s->graph_max_new = max_new; s->graph_epoch = tuning_epoch();
    return B200P_OK;
}

// Status words of a call: the session's abort word (streaming GEMMs) and the status word at the head of
// its decode workspace.  Cleared on the stream when a call starts; read back behind the call's work.
int clear_status(b200p_session* s, cudaStream_t st) {
    if (cudaError_t e = cudaMemsetAsync(s->d_abort, 0, sizeof(int), st)) return int(e);
    return int(cudaMemsetAsync(s->d_attn_status, 0, sizeof(int), st));
}
// Enqueues the read-back into words[2] (host); valid after the stream has been synchronised.
int fetch_status(b200p_session* s, int* words, cudaStream_t st) {
    if (cudaError_t e = cudaMemcpyAsync(&words[0], s->d_abort, sizeof(int), cudaMemcpyDeviceToHost, st)) return int(e);
    return int(cudaMemcpyAsync(&words[1], s->d_attn_status, sizeof(int), cudaMemcpyDeviceToHost, st));
}
int generate(b200p_session* s, const int* ids, int Tn, int max_new, int* out, float* timings, cudaStream_t st) {
    if (int e = ensure_scratch(s, Tn, max_new)) return e;
    const int B = s->batch;
    const bool use_graph = tuning(KNOB_RUNTIME_GRAPH, 1) != 0 && s->ops->graph_step(s);
    const int gemms_per_step = s->ops->gemms_per_step(s) + 1;
    cudaEvent_t e0, e1, e2;
    cudaEventCreate(&e0); cudaEventCreate(&e1); cudaEventCreate(&e2);
    int rc = B200P_OK;
    do {
        if ((rc = clear_status(s, st))) break;
        cudaEventRecord(e0, st);
        if (cudaError_t e = cudaMemcpyAsync(s->d_ids, ids, size_t(B) * Tn * sizeof(int), cudaMemcpyHostToDevice, st)) { rc = int(e); break; }
        if ((rc = embed(s, s->d_ids, B * Tn, st))) break;
        s->kv_len = 0;
        if ((rc = s->ops->run_layers(s, Tn, 0, st, nullptr))) break;
        s->kv_len = Tn;
        if ((rc = last_logits_prefill(s, Tn, st))) break;
        if ((rc = sample(s, max_new, 0, nullptr, st))) break;
        set_state_kernel<<<1, 1, 0, st>>>(s->d_state, Tn, 1);
        if ((rc = launched())) break;
        cudaEventRecord(e1, st);
        bool looped = false;
        if (max_new > 1 && s->ops->decode_loop) {
            // all remaining steps in one launch: the ids, the position and the output column stay on the device
            if (Tn + max_new - 2 >= s->max_seq) { rc = B200P_E_RANGE; break; }
            if ((rc = s->ops->decode_loop(s, s->d_next, max_new - 1, true, s->d_tokens, max_new, st, &looped))) break;
            if (looped) s->kv_len += max_new - 1;
        }
        for (int step = 1; step < max_new && !looped; ++step) {
            if (s->kv_len >= s->max_seq) { rc = B200P_E_RANGE; break; }
            if (use_graph && step >= 2) {
                // the first decode step ran eagerly below; from the second on, replay the captured step
                if (!s->step_graph || s->graph_hidden != s->hidden || s->graph_tokens != s->d_tokens || s->graph_max_new != max_new ||
                    s->graph_epoch != tuning_epoch()) {
                    if (build_step_graph(s, max_new) != B200P_OK) drop_step_graph(s);
                }
                if (s->step_graph) {
                    if (cudaError_t e = cudaGraphLaunch(s->step_graph, st)) { rc = int(e); break; }
                    s->kv_len += 1;
                    s->gemm_calls += gemms_per_step;
                    g_launches.fetch_add(s->graph_kernels, std::memory_order_relaxed);
                    ++s->graph_replays;
                    continue;
                }
            }
            if ((rc = decode_step_device_state(s, max_new, st))) break;
            s->kv_len += 1;
        }
        if (rc) break;
        cudaEventRecord(e2, st);
        if (cudaError_t e = cudaMemcpyAsync(out, s->d_tokens, size_t(B) * max_new * sizeof(int), cudaMemcpyDeviceToHost, st)) { rc = int(e); break; }
        int words[2] = {0, 0};
        if ((rc = fetch_status(s, words, st))) break;
        if (cudaError_t e = cudaStreamSynchronize(st)) { rc = int(e); break; }
        if ((rc = status_words_rc(words, 2))) break;            // a bounded wait gave up: the tokens are not to be trusted
        if (timings) { cudaEventElapsedTime(&timings[0], e0, e1); cudaEventElapsedTime(&timings[1], e1, e2); }
    } while (false);
    cudaEventDestroy(e0); cudaEventDestroy(e1); cudaEventDestroy(e2);
    return rc;
}

// Copies the status words of a call's work and waits for it.
int finish_call(b200p_session* s, cudaStream_t st) {
    int words[2] = {0, 0};
    if (int e = fetch_status(s, words, st)) return e;
    if (cudaError_t e = cudaStreamSynchronize(st)) return int(e);
    return status_words_rc(words, 2);
}

int prefill_logits(b200p_session* s, const int* ids, int Tn, float* logits, cudaStream_t st) {
    if (int e = ensure_scratch(s, Tn, 1)) return e;
    const int B = s->batch;
    if (int e = clear_status(s, st)) return e;
    if (cudaError_t e = cudaMemcpyAsync(s->d_ids, ids, size_t(B) * Tn * sizeof(int), cudaMemcpyHostToDevice, st)) return int(e);
    if (int e = embed(s, s->d_ids, B * Tn, st)) return e;
    s->kv_len = 0;
    if (int e = s->ops->run_layers(s, Tn, 0, st, nullptr)) return e;
    s->kv_len = Tn;
    if (int e = last_logits_prefill(s, Tn, st)) return e;
    if (cudaError_t e = cudaMemcpyAsync(logits, s->logits, size_t(B) * s->c.vocab_size * 4, cudaMemcpyDeviceToHost, st)) return int(e);
    return finish_call(s, st);
}

// One token per sequence on top of the cache; logits stay in s->logits.
int step_device(b200p_session* s, const int* ids, cudaStream_t st) {
    if (int e = ensure_scratch(s, 1, 1)) return e;
    if (s->kv_len >= s->max_seq) return B200P_E_RANGE;
    const int B = s->batch;
    if (cudaError_t e = cudaMemcpyAsync(s->d_ids, ids, size_t(B) * sizeof(int), cudaMemcpyHostToDevice, st)) return int(e);
    // same device-side position and split plan as the greedy loop, so that both give the same bits
    set_state_kernel<<<1, 1, 0, st>>>(s->d_state, s->kv_len, 0);
    if (int e = launched()) return e;
    bool looped = false;
    // the greedy loop's kernel for one step, logits only: same arithmetic, so both give the same bits
    if (s->ops->decode_loop)
        if (int e = s->ops->decode_loop(s, s->d_ids, 1, false, nullptr, 0, st, &looped)) return e;
    if (!looped) {
        if (int e = embed(s, s->d_ids, B, st)) return e;
        if (int e = s->ops->run_layers(s, 1, 0, st, s->d_state)) return e;
        if (int e = last_logits_step(s, st)) return e;
    }
    s->kv_len += 1;
    return B200P_OK;
}

int step_logits(b200p_session* s, const int* ids, float* logits, cudaStream_t st) {
    if (int e = clear_status(s, st)) return e;
    if (int e = step_device(s, ids, st)) return e;
    if (cudaError_t e = cudaMemcpyAsync(logits, s->logits, size_t(s->batch) * s->c.vocab_size * 4, cudaMemcpyDeviceToHost, st)) return int(e);
    return finish_call(s, st);
}

// The next Tn tokens of every sequence, logits at the wanted places (host, [B, n_want, V]).
int extend(b200p_session* s, const int* ids, int Tn, const int* want, int n_want, float* logits, cudaStream_t st) {
    const int B = s->batch, V = s->c.vocab_size;
    if (int e = clear_status(s, st)) return e;
    if (Tn > 1 && s->kv_len > 0 && !s->ops->portions) {
        // the decoder's prefill starts from an empty cache only: token by token
        std::vector<int> col(B);
        for (int t = 0; t < Tn; ++t) {
            for (int b = 0; b < B; ++b) col[b] = ids[size_t(b) * Tn + t];
            if (int e = step_device(s, col.data(), st)) return e;
            for (int w = 0; w < n_want; ++w)
                if (want[w] == t)
                    for (int b = 0; b < B; ++b)
                        if (cudaError_t e = cudaMemcpyAsync(logits + (size_t(b) * n_want + w) * V, s->logits + size_t(b) * V, size_t(V) * 4, cudaMemcpyDeviceToHost, st)) return int(e);
            if (cudaError_t e = cudaStreamSynchronize(st)) return int(e);          // col is reused
        }
        return finish_call(s, st);
    }
    if (Tn == 1) {
        if (int e = step_device(s, ids, st)) return e;
        for (int w = 0; w < n_want; ++w)
            for (int b = 0; b < B; ++b)
                if (cudaError_t e = cudaMemcpyAsync(logits + (size_t(b) * n_want + w) * V, s->logits + size_t(b) * V, size_t(V) * 4, cudaMemcpyDeviceToHost, st)) return int(e);
        return finish_call(s, st);
    }
    if (int e = ensure_scratch(s, Tn, 1)) return e;
    if (cudaError_t e = cudaMemcpyAsync(s->d_ids, ids, size_t(B) * Tn * sizeof(int), cudaMemcpyHostToDevice, st)) return int(e);
    if (int e = embed(s, s->d_ids, B * Tn, st)) return e;
    if (int e = s->ops->run_layers(s, Tn, s->kv_len, st, nullptr)) return e;
    s->kv_len += Tn;
    if (n_want > 0) {
        const int rows = B * n_want;
        if (rows > s->cap_want) {
            if (cudaError_t e = s->alloc(&s->want_logits, size_t(rows) * V * 4)) return int(e);
            if (cudaError_t e = s->alloc(&s->want_norm, size_t(rows) * s->H * 4)) return int(e);
            if (cudaError_t e = s->alloc(&s->d_want, size_t(rows) * sizeof(int))) return int(e);
            s->cap_want = rows;
        }
        if (cudaError_t e = cudaMemcpyAsync(s->d_want, want, size_t(n_want) * sizeof(int), cudaMemcpyHostToDevice, st)) return int(e);
        if (int e = final_norm_rows(s, s->want_norm, rows, Tn, 0, s->d_want, n_want, st)) return e;
        if (int e = head_rows(s, s->want_norm, s->want_logits, rows, skinny_ok(s, rows), st)) return e;
        if (cudaError_t e = cudaMemcpyAsync(logits, s->want_logits, size_t(rows) * V * 4, cudaMemcpyDeviceToHost, st)) return int(e);
    }
    return finish_call(s, st);
}

// Token ids index the embedding: an id that does not exist is an error before anything is launched.
bool ids_exist(const b200p_session* s, const int* ids, size_t n) {
    for (size_t i = 0; i < n; ++i) if (ids[i] < 0 || ids[i] >= s->c.vocab_size) return false;
    return true;
}

} // namespace
} // namespace b200p

using namespace b200p;

extern "C" b200p_session* b200p_session_open(const b200p_model* m, int dtype, int max_seq, int batch, int* status) {
    int dummy; if (!status) status = &dummy;
    *status = B200P_OK;
    if (!m) { *status = B200P_E_NULL; return nullptr; }
    if (!m->arch) {                                          // the Llama-style decoder: 16-bit, in the weights' own type
        if (dtype >= 0 && dtype != m->w.dtype) { *status = B200P_E_DTYPE; return nullptr; }
        b200p_session* (*create)(const b200p_model_weights*, int, int, int*) = llama_session_create();
        if (!create) { *status = B200P_E_OP; return nullptr; }
        return create(&m->w, max_seq, batch, status);
    }
    if (max_seq <= 0 || batch <= 0) { *status = B200P_E_LENGTH; return nullptr; }
    if (sm_count() <= 0) { *status = B200P_E_NO_DEVICE; return nullptr; }
    b200p_session* s = new b200p_session();
    s->c = m->w.cfg; s->dtype = dtype < 0 ? m->w.dtype : dtype; s->max_seq = max_seq; s->batch = batch;
    int rc = m->arch->build(s, m);
    if (!rc) rc = session_common_init(s);
    if (!rc) rc = int(cudaDeviceSynchronize());
    if (rc) { *status = rc; b200p_session_destroy(s); return nullptr; }
    return s;
}

extern "C" void b200p_session_destroy(b200p_session* s) {
    if (!s) return;
    cudaDeviceSynchronize();
    if (s->step_graph) cudaGraphExecDestroy(s->step_graph);
    if (s->capture_stream) cudaStreamDestroy(s->capture_stream);
    if (s->blas) cublasDestroy(s->blas);
    for (void* p : s->owned) cudaFree(p);
    for (void* p : s->scratch) cudaFree(p);
    delete s;
}

extern "C" int b200p_session_generate(b200p_session* s, const int* ids, int T, int max_new, int* out, float* timings,
                                      b200p_stream_t stream) {
    if (!s || !ids || !out) return B200P_E_NULL;
    if (T <= 0 || max_new <= 0 || T + max_new - 1 > s->max_seq) return B200P_E_LENGTH;
    if (!ids_exist(s, ids, size_t(s->batch) * T)) return B200P_E_RANGE;
    return generate(s, ids, T, max_new, out, timings, static_cast<cudaStream_t>(stream));
}

extern "C" int b200p_session_prefill_logits(b200p_session* s, const int* ids, int T, float* logits, b200p_stream_t stream) {
    if (!s || !ids || !logits) return B200P_E_NULL;
    if (T <= 0 || T > s->max_seq) return B200P_E_LENGTH;
    if (!ids_exist(s, ids, size_t(s->batch) * T)) return B200P_E_RANGE;
    return prefill_logits(s, ids, T, logits, static_cast<cudaStream_t>(stream));
}

extern "C" int b200p_session_step_logits(b200p_session* s, const int* ids, float* logits, b200p_stream_t stream) {
    if (!s || !ids || !logits) return B200P_E_NULL;
    if (!ids_exist(s, ids, size_t(s->batch))) return B200P_E_RANGE;
    return step_logits(s, ids, logits, static_cast<cudaStream_t>(stream));
}

extern "C" int b200p_session_extend(b200p_session* s, const int* ids, int T, const int* want, int n_want, float* logits,
                                    b200p_stream_t stream) {
    if (!s || !ids || (n_want > 0 && (!want || !logits))) return B200P_E_NULL;
    if (T <= 0 || n_want < 0 || T > s->max_seq - s->kv_len) return B200P_E_LENGTH;
    for (int i = 0; i < n_want; ++i) if (want[i] < 0 || want[i] >= T) return B200P_E_RANGE;
    if (!ids_exist(s, ids, size_t(s->batch) * T)) return B200P_E_RANGE;
    return extend(s, ids, T, want, n_want, logits, static_cast<cudaStream_t>(stream));
}

extern "C" void b200p_session_reset(b200p_session* s) { if (s) s->kv_len = 0; }

extern "C" int b200p_skinny_gemm(int dtype, int prologue, int epilogue, const void* W, const void* x16, const float* x32,
                                 const void* norm_w, void* out, int M, int N, int K, int ldx, int ldo, float eps,
                                 b200p_stream_t stream) {
    if (!W || !out) return B200P_E_NULL;
    if (dtype != B200P_F16 && dtype != B200P_BF16) return B200P_E_DTYPE;
    if (prologue == PRO_PLAIN ? !x16 : (!x32 || !norm_w)) return B200P_E_NULL;
    if (sm_count() <= 0) return B200P_E_NO_DEVICE;
    SkinnyArgs a{};
    a.W = W; a.X16 = x16; a.X32 = x32; a.norm_w = norm_w; a.out = out; a.M = M; a.N = N; a.K = K; a.ldx = ldx; a.ldo = ldo; a.eps = eps;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    auto run = [&](auto tag) -> int {
        using T = decltype(tag);
        if (prologue == PRO_RMSNORM) {
            switch (epilogue) {
                case EPI_STORE16: return launch_skinny<T, PRO_RMSNORM, EPI_STORE16>(a, st);
                case EPI_STORE32: return launch_skinny<T, PRO_RMSNORM, EPI_STORE32>(a, st);
                case EPI_SILU16:  return launch_skinny<T, PRO_RMSNORM, EPI_SILU16>(a, st);
            }
        } else if (prologue == PRO_PLAIN) {
            switch (epilogue) {
                case EPI_ACC32:   return launch_skinny<T, PRO_PLAIN, EPI_ACC32>(a, st);
                case EPI_STORE32: return launch_skinny<T, PRO_PLAIN, EPI_STORE32>(a, st);
                case EPI_GELU16:  return launch_skinny<T, PRO_PLAIN, EPI_GELU16>(a, st);
            }
        }
        return B200P_E_OP;                                   // only the combinations the decode step uses exist
    };
    return dtype == B200P_F16 ? run(__half{}) : run(__nv_bfloat16{});
}

extern "C" int b200p_session_kv_len(const b200p_session* s) { return s ? s->kv_len : -1; }
extern "C" unsigned long long b200p_session_gemm_calls(const b200p_session* s) { return s ? s->gemm_calls : 0; }
extern "C" unsigned long long b200p_session_blas_calls(const b200p_session* s) { return s ? s->blas_calls : 0; }
extern "C" unsigned long long b200p_session_graph_replays(const b200p_session* s) { return s ? s->graph_replays : 0; }
extern "C" unsigned long long b200p_session_mega_launches(const b200p_session* s) { return s ? s->mega_launches : 0; }
