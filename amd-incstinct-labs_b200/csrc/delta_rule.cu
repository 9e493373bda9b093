// ---------------------------------------------------------------------------
// delta_rule.cu -- the gated delta rule (delta.cuh).
//
// Many tokens:
//   delta_prepare   CTA = (16 tokens, query/key head): convolutions, unit vectors, the blocks' dot
//                   products, decays and steps, laid out so that a block is a few bulk copies;
//   delta_blocks    CTA = (sequence, head, 64 columns of S): walks the blocks.  A warp owns 16
//                   columns, S stays in registers (8 lanes x 4 columns x rows / 8), every 16-byte
//                   read of k or q from shared memory feeds 16 FMAs, the eight sums of a token
//                   (k and q times four columns) are reduced and scattered over the eight lanes in
//                   seven shuffles, so that afterwards a lane owns one column of one kind and the
//                   sequential triangle needs one shuffle per token;
//   delta_finish    norm and gate, and the convolutions' last inputs.
// One token: delta_step, a cluster per (sequence, head), 32 columns of S per CTA; S and the
// convolutions' history are read before the dependency wait.
// ---------------------------------------------------------------------------
#include "delta.cuh"
#include "vec_quads.cuh"
#include "dme/dme_tma.cuh"
#include "wave_primitives/wave64.cuh"
#include "b200p.h"
#include <cooperative_groups.h>
#include <type_traits>

namespace b200p {
namespace {
namespace cg = cooperative_groups;
using T16 = __nv_bfloat16;

__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float4 silu4(const float4& z) { return make_float4(silu(z.x), silu(z.y), silu(z.z), silu(z.w)); }
__device__ __forceinline__ void fma4(float4& acc, const float4& w, const float4& x) { acc.x += w.x * x.x; acc.y += w.y * x.y; acc.z += w.z * x.z; acc.w += w.w * x.w; }
__device__ __forceinline__ float dot4(const float4& x, const float4& y) { return (x.x * y.x + x.y * y.y) + (x.z * y.z + x.w * y.w); }

constexpr float kUnitEps = 1e-6f;        // added to the squared length of q and k

__device__ __forceinline__ float decay(float a, float a_log, float dt_bias) {
    const float z = a + dt_bias;
    const float sp = z > 20.f ? z : log1pf(expf(z));
    return expf(-expf(a_log) * sp);
}
__device__ __forceinline__ float step_size(float b) { return 1.f / (1.f + expf(-b)); }

// packed fp32 pairs
using F2 = unsigned long long;
__device__ __forceinline__ F2 fma2(F2 a, F2 b, F2 c) { F2 r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }
__device__ __forceinline__ F2 mul2(F2 a, F2 b) { F2 r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ F2 pair(float lo, float hi) { F2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi)); return r; }
__device__ __forceinline__ float2 unpair(F2 a) { float2 r; asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(a)); return r; }
__device__ __forceinline__ float sum2(F2 a) { const float2 r = unpair(a); return r.x + r.y; }

// ---- many tokens: preparation -------------------------------------------------------------------------------
// The convolutions' input at token t of this call (negative: of earlier calls), channels c .. c + 3.
template <typename P>
__device__ __forceinline__ float4 conv_input(const DeltaArgs& a, int b, int t, int c) {
    if (t >= 0) return load4<P>(static_cast<const P*>(a.proj) + (size_t(b) * a.Tn + t) * a.ldp + c);
    const int pos = a.pos0 + t;
    if (pos < 0) return make_float4(0.f, 0.f, 0.f, 0.f);
    return load4<float>(a.ring + (size_t(b) * a.d.taps + pos % a.d.taps) * a.d.channels() + c);
}

// put(token of the block, value) for the 16 tokens from t0 on of channels c .. c + 3; tokens past the call's give 0.
template <typename P, int TAPS, typename F>
__device__ __forceinline__ void conv_block(const DeltaArgs& a, int b, int t0, int c, F&& put) {
    const int C = a.d.channels(), taps = TAPS ? TAPS : a.d.taps;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    if constexpr (TAPS > 0) {
        float4 w[TAPS], x[kDeltaBlock + TAPS - 1];
        #pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = load4<float>(a.conv + size_t(j) * C + c);
        #pragma unroll
        for (int j = 0; j < kDeltaBlock + TAPS - 1; ++j) {
            const int t = t0 + j - (TAPS - 1);
            x[j] = t < a.Tn ? conv_input<P>(a, b, t, c) : zero;
        }
        #pragma unroll
        for (int t = 0; t < kDeltaBlock; ++t) {
            float4 acc = zero;
            #pragma unroll
            for (int j = 0; j < TAPS; ++j) fma4(acc, w[j], x[t + j]);
            put(t, t0 + t < a.Tn ? silu4(acc) : zero);
        }
    } else {
        for (int t = 0; t < kDeltaBlock; ++t) {
            float4 acc = zero;
            if (t0 + t < a.Tn)
                for (int j = 0; j < taps; ++j) fma4(acc, load4<float>(a.conv + size_t(j) * C + c), conv_input<P>(a, b, t0 + t - (taps - 1) + j, c));
            put(t, silu4(acc));
        }
    }
}

template <typename P, int TAPS>
__global__ void __launch_bounds__(256) delta_prepare_kernel(const DeltaArgs a) {
    extern __shared__ __align__(16) float prep_smem[];
    const DeltaDims& d = a.d;
    const int R = d.rows(), ld = R + 4;                           // rows 16 bytes longer: 16-byte reads of different tokens on different banks
    float *ks = prep_smem, *qs = ks + kDeltaBlock * ld;           // [16][ld]
    const int blk = blockIdx.x, nblk = gridDim.x, kvh = blockIdx.y, b = blockIdx.z, t0 = blk * kDeltaBlock;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int qk_quads = R / 4, v_quads = d.slices() * 16, jobs = 2 * qk_quads + d.group() * v_quads;
    for (int job = threadIdx.x; job < jobs; job += 256) {
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        if (job < 2 * qk_quads) {
            const bool is_k = job >= qk_quads;
            const int col = 4 * (job % qk_quads);
            float* dst = (is_k ? ks : qs) + col;
            auto put = [&](int t, const float4& v) { store4<float>(dst + t * ld, v); };
            if (col < d.dim) conv_block<P, TAPS>(a, b, t0, (is_k ? d.kv_heads * d.dim : 0) + kvh * d.dim + col, put);
            else for (int t = 0; t < kDeltaBlock; ++t) put(t, zero);
        } else {
            const int i = job - 2 * qk_quads, h = kvh * d.group() + i / v_quads, col = 4 * (i % v_quads);
            float* dst = a.v + (((size_t(b) * d.heads + h) * d.slices() + col / 64) * nblk + blk) * 1024 + col % 64;
            auto put = [&](int t, const float4& v) { store4<float>(dst + t * 64, v); };
            if (col < d.vdim) conv_block<P, TAPS>(a, b, t0, 2 * d.kv_heads * d.dim + h * d.vdim + col, put);
            else for (int t = 0; t < kDeltaBlock; ++t) put(t, zero);
        }
    }
    for (int i = threadIdx.x; i < d.group() * kDeltaBlock; i += 256) {
        const int h = kvh * d.group() + i / kDeltaBlock, t = i % kDeltaBlock;
        float g = 1.f, beta = 0.f;                                // tokens past the call's leave S as it is
        if (t0 + t < a.Tn) {
            const float* ab = a.ab + (size_t(b) * a.Tn + t0 + t) * a.ld_ab;
            g = decay(ab[h], a.a_log[h], a.dt_bias[h]);
            beta = step_size(ab[d.heads + h]);
        }
        float* dst = a.gb + ((size_t(b) * d.heads + h) * nblk + blk) * 32 + t;
        dst[0] = g; dst[16] = beta;
    }
    __syncthreads();
    float* out = a.kq + ((size_t(b) * d.kv_heads + kvh) * nblk + blk) * d.kq_block();
    const float q_scale = rsqrtf(float(d.n_dim));
    for (int t = warp; t < 2 * kDeltaBlock; t += 8) {             // unit vectors: 16 keys, then 16 queries
        float* row = (t < kDeltaBlock ? ks : qs - kDeltaBlock * ld) + t * ld;
        float ss = 0.f;
        for (int c = 4 * lane; c < R; c += 128) { const float4 v = load4<float>(row + c); ss += dot4(v, v); }
        const float f = rsqrtf(wave::dpp::reduce_sum(ss) + kUnitEps) * (t < kDeltaBlock ? 1.f : q_scale);
        for (int c = 4 * lane; c < R; c += 128) {
            const float4 v = load4<float>(row + c), s = make_float4(v.x * f, v.y * f, v.z * f, v.w * f);
            store4<float>(row + c, s);
            store4<float>(out + size_t(t) * R + c, s);
        }
    }
    __syncthreads();
    const int i = threadIdx.x / 16, t = threadIdx.x % 16;
    float kk = 0.f, kq = 0.f;
    if (t >= i)
        for (int c = 0; c < R; c += 4) {
            const float4 x = load4<float>(ks + i * ld + c);
            kk += dot4(x, load4<float>(ks + t * ld + c));
            kq += dot4(x, load4<float>(qs + t * ld + c));
        }
    out[32 * R + threadIdx.x] = kk;
    out[32 * R + 256 + threadIdx.x] = kq;
}

// ---- many tokens: the blocks ----------------------------------------------------------------------------------
constexpr int kBlockThreads = 128, kBlockStages = 2;
template <int DL> struct BlockSmem {                              // floats; DL rows of S per lane
    static constexpr int R = 8 * DL, KQ = 32 * R + 512, OFF_V = KQ, OFF_GB = KQ + 1024, STAGE = OFF_GB + 32;
    static constexpr int OFF_MX = kBlockStages * STAGE;           // [2][2 kinds][16 i][16 t], then [2][G 16 | R_t16 16]
    static constexpr int OFF_G = OFF_MX + 2 * 512, OFF_U = OFF_G + 2 * 32, FLOATS = OFF_U + 4 * 256;
    static constexpr int BYTES = FLOATS * 4 + 64;
};

template <int DL>
__global__ void __launch_bounds__(kBlockThreads) delta_blocks_kernel(const DeltaArgs a, int* sticky) {
    using Sh = BlockSmem<DL>;
    constexpr int R = Sh::R, ST = kBlockStages;
    extern __shared__ __align__(128) float blk_smem[];
    uint64_t* full = reinterpret_cast<uint64_t*>(blk_smem + Sh::FLOATS);
    const DeltaDims& d = a.d;
    const int slice = blockIdx.x, h = blockIdx.y, b = blockIdx.z, kvh = h / d.group();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, grp = lane / 8, j = lane % 8;
    const int nblk = (a.Tn + kDeltaBlock - 1) / kDeltaBlock;
    const float* src_kq = a.kq + (size_t(b) * d.kv_heads + kvh) * nblk * d.kq_block();
    const float* src_v = a.v + ((size_t(b) * d.heads + h) * d.slices() + slice) * nblk * 1024;
    const float* src_gb = a.gb + (size_t(b) * d.heads + h) * nblk * 32;
    if (threadIdx.x == 0) {
        for (int s = 0; s < ST; ++s) dme::mbar_init(&full[s], 1);
        dme::mbar_init_fence();
    }
    __syncthreads();
    auto fetch = [&](int n) {                                     // one thread: block n into its stage
        float* dst = blk_smem + (n % ST) * Sh::STAGE;
        dme::mbar_arrive_expect_tx(&full[n % ST], Sh::STAGE * 4);
        dme::copy_tile_1d(dst, src_kq + size_t(n) * Sh::KQ, Sh::KQ * 4, &full[n % ST]);
        dme::copy_tile_1d(dst + Sh::OFF_V, src_v + size_t(n) * 1024, 4096, &full[n % ST]);
        dme::copy_tile_1d(dst + Sh::OFF_GB, src_gb + size_t(n) * 32, 128, &full[n % ST]);
    };
    if (threadIdx.x == 0) for (int n = 0; n < ST && n < nblk; ++n) fetch(n);

    // S: columns col0 .. col0 + 3, rows 32 x + 4 j .. + 3
    const int wcol = slice * 64 + warp * 16, col0 = wcol + grp * 4;
    const bool kind_q = (j & 4) != 0;                             // after the reduction: which product, and of which column
    const int mycol = grp * 4 + (j & 3);                          // in the warp's 16
    float* state = a.state + (size_t(b) * d.heads + h) * R * d.vdim;
    F2 S[4][DL / 2];
    #pragma unroll
    for (int p = 0; p < DL / 2; ++p) {
        const int r = 32 * (p / 2) + 4 * j + 2 * (p % 2);
        #pragma unroll
        for (int c = 0; c < 4; ++c) {
            const bool live = a.pos0 > 0 && col0 + c < d.vdim;
            S[c][p] = live ? pair(state[size_t(r) * d.vdim + col0 + c], state[size_t(r + 1) * d.vdim + col0 + c]) : 0ull;
        }
    }
    float* U = blk_smem + Sh::OFF_U + warp * 256;                 // [16 t][16 columns] of this warp
    bool ok = true;
    for (int n = 0; n < nblk; ++n) {
        ok = dme::wait(&full[n % ST], uint32_t((n / ST) & 1), a.abort_word);
        const float* st = blk_smem + (n % ST) * Sh::STAGE;
        const float* g = st + Sh::OFF_GB;
        float* mx = blk_smem + Sh::OFF_MX + (n & 1) * 512;
        float* G = blk_smem + Sh::OFF_G + (n & 1) * 32;
        if (ok) {
            // the triangle's factors, with the decays between the two tokens
            const int i = threadIdx.x / 8, t = 2 * (threadIdx.x % 8);
            float r = 1.f;
            for (int x = i + 1; x <= t; ++x) r *= g[x];
            const float* dots = st + 32 * R + i * 16 + t;
            const float2 kk = *reinterpret_cast<const float2*>(dots), kq = *reinterpret_cast<const float2*>(dots + 256);
            const float f0 = r, f1 = i <= t ? r * g[t + 1] : 1.f;
            *reinterpret_cast<float2*>(mx + i * 16 + t) = make_float2(t > i ? -kk.x * f0 : 0.f, t + 1 > i ? -kk.y * f1 : 0.f);
            *reinterpret_cast<float2*>(mx + 256 + i * 16 + t) = make_float2(t >= i ? kq.x * f0 : 0.f, t + 1 >= i ? kq.y * f1 : 0.f);
            if (threadIdx.x < 32) {
                const int y = threadIdx.x % 16;
                float f = 1.f;
                if (threadIdx.x < 16) for (int x = 0; x <= y; ++x) f *= g[x];
                else                  for (int x = y + 1; x < 16; ++x) f *= g[x];
                G[threadIdx.x] = f;
            }
        }
        // every warp is past block n - 1 here, so its stage can be filled again
        if (!__syncthreads_and(ok)) { ok = false; break; }
        if (threadIdx.x == 0 && n >= 1 && n - 1 + ST < nblk) fetch(n - 1 + ST);
        // ---- products with S: k and q of every token, four columns ------------------------------------------------
        float acc[kDeltaBlock];
        #pragma unroll
        for (int t = 0; t < kDeltaBlock; ++t) {
            F2 ak[4] = {0ull, 0ull, 0ull, 0ull}, aq[4] = {0ull, 0ull, 0ull, 0ull};
            #pragma unroll
            for (int x = 0; x < DL / 4; ++x) {
                const ulonglong2 kv = *reinterpret_cast<const ulonglong2*>(st + t * R + 32 * x + 4 * j);
                const ulonglong2 qv = *reinterpret_cast<const ulonglong2*>(st + (16 + t) * R + 32 * x + 4 * j);
                #pragma unroll
                for (int c = 0; c < 4; ++c) {
                    ak[c] = fma2(S[c][2 * x], kv.x, ak[c]); ak[c] = fma2(S[c][2 * x + 1], kv.y, ak[c]);
                    aq[c] = fma2(S[c][2 * x], qv.x, aq[c]); aq[c] = fma2(S[c][2 * x + 1], qv.y, aq[c]);
                }
            }
            float r4[4], r2[2];
            #pragma unroll
            for (int c = 0; c < 4; ++c) {
                const float sk = sum2(ak[c]), sq = sum2(aq[c]);
                r4[c] = (kind_q ? sq : sk) + __shfl_xor_sync(0xffffffffu, kind_q ? sk : sq, 4);
            }
            #pragma unroll
            for (int c = 0; c < 2; ++c) r2[c] = ((j & 2) ? r4[2 + c] : r4[c]) + __shfl_xor_sync(0xffffffffu, (j & 2) ? r4[c] : r4[2 + c], 2);
            const float r1 = ((j & 1) ? r2[1] : r2[0]) + __shfl_xor_sync(0xffffffffu, (j & 1) ? r2[0] : r2[1], 1);
            acc[t] = G[t] * (kind_q ? r1 : -r1);
        }
        if (!kind_q) {
            #pragma unroll
            for (int t = 0; t < kDeltaBlock; ++t) acc[t] += st[Sh::OFF_V + t * 64 + warp * 16 + mycol];
        }
        // ---- the triangle: lanes of k find u_t one after the other, lanes of q gather the outputs ------------------
        const float* m = mx + (kind_q ? 256 : 0);
        #pragma unroll
        for (int i = 0; i < kDeltaBlock; ++i) {
            const float u = __shfl_sync(0xffffffffu, acc[i] * g[16 + i], lane & ~4);
            if (!kind_q) U[i * 16 + mycol] = u * G[16 + i];
            #pragma unroll
            for (int t4 = i / 4 * 4; t4 < kDeltaBlock; t4 += 4) {
                const float4 f = load4<float>(m + i * 16 + t4);
                if (t4 + 0 >= i) acc[t4 + 0] += f.x * u;
                if (t4 + 1 >= i) acc[t4 + 1] += f.y * u;
                if (t4 + 2 >= i) acc[t4 + 2] += f.z * u;
                acc[t4 + 3] += f.w * u;
            }
        }
        if (kind_q && wcol + mycol < d.vdim) {
            float* o = a.o + (size_t(b) * a.Tn + n * kDeltaBlock) * d.v_row() + size_t(h) * d.vdim + wcol + mycol;
            #pragma unroll
            for (int t = 0; t < kDeltaBlock; ++t) if (n * kDeltaBlock + t < a.Tn) o[size_t(t) * d.v_row()] = acc[t];
        }
        __syncwarp();
        // ---- the update -----------------------------------------------------------------------------------------
        const F2 g16 = pair(G[15], G[15]);
        #pragma unroll
        for (int c = 0; c < 4; ++c)
            #pragma unroll
            for (int p = 0; p < DL / 2; ++p) S[c][p] = mul2(S[c][p], g16);
        #pragma unroll 4
        for (int t = 0; t < kDeltaBlock; ++t) {
            const float4 u = load4<float>(U + t * 16 + grp * 4);
            const F2 up[4] = {pair(u.x, u.x), pair(u.y, u.y), pair(u.z, u.z), pair(u.w, u.w)};
            #pragma unroll
            for (int x = 0; x < DL / 4; ++x) {
                const ulonglong2 kv = *reinterpret_cast<const ulonglong2*>(st + t * R + 32 * x + 4 * j);
                #pragma unroll
                for (int c = 0; c < 4; ++c) { S[c][2 * x] = fma2(kv.x, up[c], S[c][2 * x]); S[c][2 * x + 1] = fma2(kv.y, up[c], S[c][2 * x + 1]); }
            }
        }
        __syncwarp();                                             // U is read before the next block writes it
    }
    if (!ok) { if (threadIdx.x == 0) { atomicExch(a.abort_word, 1); atomicExch(sticky, 1); } return; }
    #pragma unroll
    for (int p = 0; p < DL / 2; ++p) {
        const int r = 32 * (p / 2) + 4 * j + 2 * (p % 2);
        #pragma unroll
        for (int c = 0; c < 4; ++c)
            if (col0 + c < d.vdim) {
                const float2 v = unpair(S[c][p]);
                state[size_t(r) * d.vdim + col0 + c] = v.x; state[size_t(r + 1) * d.vdim + col0 + c] = v.y;
            }
    }
}

// Token by token, any size: one warp per column of S, rows lane, lane + 32, ...
template <int NR>
__global__ void __launch_bounds__(256) delta_plain_kernel(const DeltaArgs a) {
    const DeltaDims& d = a.d;
    const int R = d.rows(), warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int col = blockIdx.x * 8 + warp, h = blockIdx.y, b = blockIdx.z;
    if (col >= d.vdim) return;
    const int nblk = (a.Tn + kDeltaBlock - 1) / kDeltaBlock;
    const float* kq = a.kq + (size_t(b) * d.kv_heads + h / d.group()) * nblk * d.kq_block();
    const float* v = a.v + ((size_t(b) * d.heads + h) * d.slices() + col / 64) * nblk * 1024 + col % 64;
    const float* gb = a.gb + (size_t(b) * d.heads + h) * nblk * 32;
    float* state = a.state + (size_t(b) * d.heads + h) * R * d.vdim + col;
    float S[NR];
    #pragma unroll
    for (int i = 0; i < NR; ++i) { const int r = lane + 32 * i; S[i] = a.pos0 > 0 && r < R ? state[size_t(r) * d.vdim] : 0.f; }
    for (int t = 0; t < a.Tn; ++t) {
        const int n = t / kDeltaBlock, x = t % kDeltaBlock;
        const float *k = kq + size_t(n) * d.kq_block() + x * R, *q = k + 16 * R;
        const float g = gb[n * 32 + x], beta = gb[n * 32 + 16 + x];
        float kr[NR], p = 0.f, o = 0.f;
        #pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int r = lane + 32 * i;
            kr[i] = r < R ? k[r] : 0.f;
            S[i] *= g;
            p += S[i] * kr[i];
        }
        const float u = beta * (v[size_t(n) * 1024 + x * 64] - wave::dpp::reduce_sum(p));
        #pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int r = lane + 32 * i;
            S[i] += kr[i] * u;
            if (r < R) o += S[i] * q[r];
        }
        o = wave::dpp::reduce_sum(o);
        if (lane == 0) a.o[(size_t(b) * a.Tn + t) * d.v_row() + size_t(h) * d.vdim + col] = o;
    }
    #pragma unroll
    for (int i = 0; i < NR; ++i) { const int r = lane + 32 * i; if (r < R) state[size_t(r) * d.vdim] = S[i]; }
}

// ---- many tokens: norm and gate, one warp per (token, head); further warps keep the convolutions' last inputs ------
template <typename T, typename P>
__global__ void __launch_bounds__(256) delta_finish_kernel(const DeltaArgs a) {
    const DeltaDims& d = a.d;
    const size_t j = size_t(blockIdx.x) * 8 + threadIdx.x / 32, jobs = size_t(a.batch) * a.Tn * d.heads;
    const int lane = threadIdx.x % 32;
    if (j >= jobs) {
        const size_t i = j - jobs;                                // (sequence, one of the last tokens)
        const int keep = min(d.taps, a.Tn);
        if (i >= size_t(a.batch) * keep) return;
        const int b = int(i / keep), t = a.Tn - 1 - int(i % keep);
        float* dst = a.ring + (size_t(b) * d.taps + (a.pos0 + t) % d.taps) * d.channels();
        for (int c = 4 * lane; c < d.channels(); c += 128) store4<float>(dst + c, conv_input<P>(a, b, t, c));
        return;
    }
    const size_t row = j / d.heads;
    const int h = int(j % d.heads);
    const float* o = a.o + row * d.v_row() + size_t(h) * d.vdim;
    const P* gate = static_cast<const P*>(a.proj) + row * a.ldp + d.g_col() + size_t(h) * d.vdim;
    T* out = static_cast<T*>(a.out) + row * d.v_row() + size_t(h) * d.vdim;
    float ss = 0.f;
    for (int c = 4 * lane; c < d.vdim; c += 128) { const float4 v = load4<float>(o + c); ss += dot4(v, v); }
    const float f = rsqrtf(wave::dpp::reduce_sum(ss) / d.n_vdim + a.eps);
    for (int c = 4 * lane; c < d.vdim; c += 128) {
        const float4 v = load4<float>(o + c), w = load4<float>(a.norm + c), s = silu4(load4<P>(gate + c));
        store4<T>(out + c, make_float4(v.x * f * w.x * s.x, v.y * f * w.y * s.y, v.z * f * w.z * s.z, v.w * f * w.w * s.w));
    }
}

// ---- one token --------------------------------------------------------------------------------------------------
constexpr int kStepThreads = 256, kStepWarps = 8, kStepCols = 32, kStepMaxSlices = 8;

// DR rows of S per thread: rows warp, warp + 8, ...; column = lane.
template <typename T, typename P, int DR>
__global__ void __launch_bounds__(kStepThreads) delta_step_kernel(const DeltaArgs a) {
    griddep_launch_dependents();
    constexpr int R = 8 * DR;
    __shared__ __align__(16) float xs[2 * R + kStepCols];         // q, k, v after the convolutions (not yet unit vectors)
    __shared__ float red[2][kStepWarps][kStepCols];
    __shared__ float scal[5];                                     // |q|^2, |k|^2, q.k, decay, step
    __shared__ float ss_all[kStepMaxSlices];
    cg::cluster_group cluster = cg::this_cluster();
    cluster.barrier_arrive();                                     // peers run: their shared memory may be written
    const DeltaDims& d = a.d;
    const int slice = blockIdx.x, h = blockIdx.y, b = blockIdx.z, kvh = h / d.group();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, col = slice * kStepCols + lane;
    const bool live = col < d.vdim;
    const int pos = a.pos_dev ? min(*a.pos_dev, a.max_seq - 1) : a.pos0;
    float* state = a.state + (size_t(b) * d.heads + h) * R * d.vdim + col;
    float S[DR];
    #pragma unroll
    for (int i = 0; i < DR; ++i) S[i] = live && pos > 0 ? state[size_t(warp + 8 * i) * d.vdim] : 0.f;
    // the convolutions up to the current token's tap; a thread has at most two channels
    const int C = d.channels();
    int chan[2]; float part[2], w0[2];
    #pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int i = threadIdx.x + kStepThreads * x;
        chan[x] = -1; part[x] = 0.f; w0[x] = 0.f;
        if (i < 2 * R) { const int c = i % R; if (c < d.dim) chan[x] = (i < R ? 0 : d.kv_heads * d.dim) + kvh * d.dim + c; }
        else if (i < 2 * R + kStepCols) { const int c = slice * kStepCols + i - 2 * R; if (c < d.vdim) chan[x] = 2 * d.kv_heads * d.dim + h * d.vdim + c; }
        if (chan[x] >= 0) {
            w0[x] = a.conv[size_t(d.taps - 1) * C + chan[x]];
            for (int t = 1; t < d.taps && t <= pos; ++t)
                part[x] += a.conv[size_t(d.taps - 1 - t) * C + chan[x]] * a.ring[(size_t(b) * d.taps + (pos - t) % d.taps) * C + chan[x]];
        }
    }
    griddep_wait();
    const P* p = static_cast<const P*>(a.proj) + size_t(b) * a.ldp;
    float gate = 0.f, norm = 0.f;
    if (warp == 0 && live) { gate = to_float(p[d.g_col() + size_t(h) * d.vdim + col]); norm = a.norm[col]; }
    #pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int i = threadIdx.x + kStepThreads * x;
        if (i < 2 * R + kStepCols) {
            float v = 0.f;
            if (chan[x] >= 0) {
                const float in = to_float(p[chan[x]]);
                v = silu(part[x] + w0[x] * in);
                // a ring of `taps` slots: the current token's is not among those that are read in this step
                if (i >= 2 * R || (slice == 0 && h % d.group() == 0)) a.ring[(size_t(b) * d.taps + pos % d.taps) * C + chan[x]] = in;
            }
            xs[i] = v;
        }
    }
    __syncthreads();
    const float *xq = xs, *xk = xs + R, *xv = xs + 2 * R;
    if (warp < 3) {
        float s = 0.f;
        for (int c = lane; c < R; c += 32) s += (warp == 1 ? xk[c] : xq[c]) * (warp == 0 ? xq[c] : xk[c]);
        s = wave::dpp::reduce_sum(s);
        if (lane == 0) scal[warp] = s;
    } else if (warp == 3 && lane == 0) {
        const float* ab = a.ab + size_t(b) * a.ld_ab;
        scal[3] = decay(ab[h], a.a_log[h], a.dt_bias[h]);
        scal[4] = step_size(ab[d.heads + h]);
    }
    float pk = 0.f, pq = 0.f;
    #pragma unroll
    for (int i = 0; i < DR; ++i) { pk += S[i] * xk[warp + 8 * i]; pq += S[i] * xq[warp + 8 * i]; }
    red[0][warp][lane] = pk; red[1][warp][lane] = pq;
    __syncthreads();
    pk = pq = 0.f;
    #pragma unroll
    for (int w = 0; w < kStepWarps; ++w) { pk += red[0][w][lane]; pq += red[1][w][lane]; }
    const float g = scal[3], rk = rsqrtf(scal[1] + kUnitEps), rq = rsqrtf(scal[0] + kUnitEps) * rsqrtf(float(d.n_dim));
    const float u = scal[4] * (xv[lane] - g * pk * rk);
    if (live) {
        #pragma unroll
        for (int i = 0; i < DR; ++i) state[size_t(warp + 8 * i) * d.vdim] = g * S[i] + xk[warp + 8 * i] * rk * u;
    }
    const float o = g * pq * rq + u * (scal[2] * rq * rk);        // (g S + k u^T)^T q
    const float ss = wave::dpp::reduce_sum(live ? o * o : 0.f);
    cluster.barrier_wait();
    const int slices = gridDim.x;
    if (warp == 0 && lane < slices) cluster.map_shared_rank(ss_all, lane)[slice] = ss;
    cluster.sync();
    if (warp == 0 && live) {
        float tot = 0.f;
        for (int s = 0; s < slices; ++s) tot += ss_all[s];
        static_cast<T*>(a.out)[size_t(b) * d.v_row() + size_t(h) * d.vdim + col] = from_float<T>(o * rsqrtf(tot / d.n_vdim + a.eps) * norm * silu(gate));
    }
}

template <typename T, typename P>
int launch_step(const DeltaArgs& a, cudaStream_t st) {
    const int slices = (a.d.vdim + kStepCols - 1) / kStepCols;
    const dim3 grid(unsigned(slices), unsigned(a.d.heads), unsigned(a.batch));
    switch (a.d.rows() / 32) {
        case 1: return launch_dependent_clusters(delta_step_kernel<T, P, 4>, slices, grid, kStepThreads, 0, st, a);
        case 2: return launch_dependent_clusters(delta_step_kernel<T, P, 8>, slices, grid, kStepThreads, 0, st, a);
        case 3: return launch_dependent_clusters(delta_step_kernel<T, P, 12>, slices, grid, kStepThreads, 0, st, a);
        case 4: return launch_dependent_clusters(delta_step_kernel<T, P, 16>, slices, grid, kStepThreads, 0, st, a);
    }
    return B200P_E_RANGE;
}

template <int DL>
int launch_blocks(const DeltaArgs& a, cudaStream_t st) {
    using Sh = BlockSmem<DL>;
    int* sticky = device_status_ptr();
    if (!sticky) return B200P_E_NO_DEVICE;
    auto kern = delta_blocks_kernel<DL>;
    if (cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::BYTES)) return int(e);
    kern<<<dim3(unsigned(a.d.slices()), unsigned(a.d.heads), unsigned(a.batch)), kBlockThreads, Sh::BYTES, st>>>(a, sticky);
    return launched();
}

template <typename P>
int launch_prepare(const DeltaArgs& a, int nblk, cudaStream_t st) {
    const size_t smem = size_t(2) * kDeltaBlock * (a.d.rows() + 4) * 4;
    auto kern = a.d.taps == 4 ? delta_prepare_kernel<P, 4> : delta_prepare_kernel<P, 0>;
    if (smem > 48 * 1024)
        if (cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem))) return int(e);
    kern<<<dim3(unsigned(nblk), unsigned(a.d.kv_heads), unsigned(a.batch)), 256, smem, st>>>(a);
    return launched();
}

} // namespace

bool delta_step_ok(const DeltaDims& d) { return d.rows() <= 128 && d.vdim <= kStepCols * kStepMaxSlices && d.heads <= 65535; }

int delta_step(const DeltaArgs& a, cudaStream_t st) {
    if (!delta_step_ok(a.d) || a.Tn != 1 || a.batch > 65535) return B200P_E_RANGE;
    if (a.dtype == B200P_F32) return launch_step<float, float>(a, st);
    return a.proj_dtype == B200P_F32 ? launch_step<T16, float>(a, st) : launch_step<T16, T16>(a, st);
}

int delta_tokens(const DeltaArgs& a, cudaStream_t st) {
    const DeltaDims& d = a.d;
    if (d.rows() > 512) return B200P_E_DIM;
    if (d.heads > 65535 || a.batch > 65535) return B200P_E_RANGE;
    const bool f32 = a.proj_dtype == B200P_F32;
    const int nblk = (a.Tn + kDeltaBlock - 1) / kDeltaBlock;
    if (int e = f32 ? launch_prepare<float>(a, nblk, st) : launch_prepare<T16>(a, nblk, st)) return e;
    int rc;
    if (d.rows() <= 128 && tuning(KNOB_DELTA_PLAIN, 0) == 0) {
        rc = d.rows() <= 32 ? launch_blocks<4>(a, st) : d.rows() <= 64 ? launch_blocks<8>(a, st) : d.rows() <= 96 ? launch_blocks<12>(a, st) : launch_blocks<16>(a, st);
    } else {
        const dim3 grid(unsigned((d.vdim + 7) / 8), unsigned(d.heads), unsigned(a.batch));
        if (d.rows() <= 128) delta_plain_kernel<4><<<grid, 256, 0, st>>>(a);
        else delta_plain_kernel<16><<<grid, 256, 0, st>>>(a);
        rc = launched();
    }
    if (rc) return rc;
    const size_t warps = size_t(a.batch) * a.Tn * d.heads + size_t(a.batch) * (d.taps < a.Tn ? d.taps : a.Tn);
    const unsigned fin = unsigned((warps + 7) / 8);
    if (a.dtype == B200P_F32) delta_finish_kernel<float, float><<<fin, 256, 0, st>>>(a);
    else if (f32) delta_finish_kernel<T16, float><<<fin, 256, 0, st>>>(a);
    else delta_finish_kernel<T16, T16><<<fin, 256, 0, st>>>(a);
    return launched();
}

} // namespace b200p
