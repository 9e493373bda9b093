// ---------------------------------------------------------------------------
// delta_rule.cu -- the gated delta rule (delta.cuh).
//
// Many tokens:
//   delta_prepare   CTA = (16 tokens, query/key head), all in parallel: convolutions, unit vectors, the
//                   blocks' dot products, and per head the block form's matrices, laid out so that a
//                   block is a few bulk copies;
//   delta_blocks    CTA = (sequence, head, 16 to 64 columns of S): walks the blocks.  S stays in
//                   registers, the rows come through a ring of bulk copies;
//   delta_finish    norm and gate, and the convolutions' last inputs.
// Preparation and walk come in two forms.  16-bit sessions run the products on the tensor cores
// (the _mma kernels): three tf32 passes per product with fp32 accumulation, relative error of a product
// about 2^-21.  fp32 sessions run them as packed fp32x2 FMAs: S over 8 lanes x rows / 8 with 1 to 4 columns
// per lane, eight sums at a time reduced and scattered over the eight lanes in seven shuffles; a lane's
// loads from shared memory, one word per column and FMA, bound that form.
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

// FAST: on the SFU, for activations that become 16-bit operands or belong to the convolutions
template <bool FAST = false> __device__ __forceinline__ float silu(float z) { return FAST ? __fdividef(z, 1.f + __expf(-z)) : z / (1.f + expf(-z)); }
template <bool FAST = false> __device__ __forceinline__ float4 silu4(const float4& z) { return make_float4(silu<FAST>(z.x), silu<FAST>(z.y), silu<FAST>(z.z), silu<FAST>(z.w)); }
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

// fp32 products on the tensor cores: an operand is split into a tf32 number and the rest, and three of the four partial
// products are summed in fp32 (the fourth is below 2^-20 of the product).
struct Split { uint32_t hi, lo; };
__device__ __forceinline__ Split split(float x) {
    const uint32_t hi = __float_as_uint(x) & 0xffffe000u;
    return {hi, __float_as_uint(x - __uint_as_float(hi))};
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// D(16x8) += A(16x8) B(8x8): lane (r = lane / 4, q = lane % 4) holds A[r][q], A[r+8][q], A[r][q+4], A[r+8][q+4],
// B[q][r], B[q+4][r] and D[r][2q], D[r][2q+1], D[r+8][2q], D[r+8][2q+1].
__device__ __forceinline__ void mma_fp32(float (&d)[4], const Split (&a)[4], const Split& b0, const Split& b1) {
    mma_tf32(d, a[0].lo, a[1].lo, a[2].lo, a[3].lo, b0.hi, b1.hi);
    mma_tf32(d, a[0].hi, a[1].hi, a[2].hi, a[3].hi, b0.lo, b1.lo);
    mma_tf32(d, a[0].hi, a[1].hi, a[2].hi, a[3].hi, b0.hi, b1.hi);
}

// ---- many tokens: preparation -------------------------------------------------------------------------------
// The convolutions' input at token t of this call (negative: of earlier calls), channels c .. c + 3.
template <typename P>
__device__ __forceinline__ float4 conv_input(const DeltaArgs& a, int b, int t, int c) {
    if (t >= 0) return load4<P>(static_cast<const P*>(a.proj) + (size_t(b) * a.Tn + t) * a.ldp + c);
    const int pos = a.pos0 + t;
    if (pos < 0) return make_float4(0.f, 0.f, 0.f, 0.f);
    return load4<float>(a.ring + (size_t(b) * a.d.taps + pos % a.d.taps) * a.d.channels() + c);
}

// put(token of the block, value) for four tokens from t0 + tq on of channels c .. c + 3; tokens past the call's give 0.
template <typename P, int TAPS, bool FAST = false, typename F>
__device__ __forceinline__ void conv_tokens(const DeltaArgs& a, int b, int t0, int tq, int c, F&& put) {
    const int C = a.d.channels();
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    if constexpr (TAPS > 0) {
        float4 w[TAPS], x[4 + TAPS - 1];
        #pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = load4<float>(a.conv + size_t(j) * C + c);
        if (t0 >= TAPS - 1 && t0 + kDeltaBlock <= a.Tn) {         // the whole block and its history are tokens of this call
            const P* src = static_cast<const P*>(a.proj) + (size_t(b) * a.Tn + t0 + tq - (TAPS - 1)) * a.ldp + c;
            #pragma unroll
            for (int j = 0; j < 4 + TAPS - 1; ++j) x[j] = load4<P>(src + size_t(j) * a.ldp);
        } else {
            #pragma unroll
            for (int j = 0; j < 4 + TAPS - 1; ++j) {
                const int t = t0 + tq + j - (TAPS - 1);
                x[j] = t < a.Tn ? conv_input<P>(a, b, t, c) : zero;
            }
        }
        #pragma unroll
        for (int t = 0; t < 4; ++t) {
            float4 acc = zero;
            #pragma unroll
            for (int j = 0; j < TAPS; ++j) fma4(acc, w[j], x[t + j]);
            put(tq + t, t0 + tq + t < a.Tn ? silu4<FAST>(acc) : zero);
        }
    } else {
        for (int t = tq; t < tq + 4; ++t) {
            float4 acc = zero;
            if (t0 + t < a.Tn)
                for (int j = 0; j < a.d.taps; ++j) fma4(acc, load4<float>(a.conv + size_t(j) * C + c), conv_input<P>(a, b, t0 + t - (a.d.taps - 1) + j, c));
            put(t, silu4<FAST>(acc));
        }
    }
}

// Floats of the preparation's shared memory beside the rows of k, q and v.
struct PrepMatrices {
    float kk[256], kq[256];            // (k_i.k_t), (k_i.q_t) at [i][t]
    float l[256], m[256];              // the triangles of u and o at [t][i]
    float t_[256], mt[256];            // T and M T at [j][t]
    float tg[256], mtg[256];           // the same with the decay from the block's start to j
    float g[16], beta[16], G[16], tail[16];
};

// PLAIN: k, q, v, decays and steps as they are (delta_plain_kernel), no block form.
template <typename P, int TAPS, bool PLAIN>
__global__ void __launch_bounds__(256) delta_prepare_kernel(const DeltaArgs a) {
    extern __shared__ __align__(16) float prep_smem[];
    __shared__ __align__(16) PrepMatrices x;
    const DeltaDims& d = a.d;
    const int R = d.rows(), ld = R + 4, ldv = d.vdim + 4;         // rows 16 bytes longer: 16-byte reads of different tokens on different banks
    float *ks = prep_smem, *qs = ks + kDeltaBlock * ld, *vs = qs + kDeltaBlock * ld;
    const int blk = blockIdx.x, nblk = gridDim.x, kvh = blockIdx.y, b = blockIdx.z, t0 = blk * kDeltaBlock;
    const int tid = threadIdx.x, warp = tid / 32, lane = tid % 32;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int job = tid; job < 2 * R; job += 256) {                // (q or k, columns, four tokens)
        const int quad = job % (R / 4), tq = job / (R / 4) % 4 * 4, col = 4 * quad;
        const bool is_k = job >= R;
        float* dst = (is_k ? ks : qs) + col;
        auto put = [&](int t, const float4& v) { store4<float>(dst + t * ld, v); };
        if (col < d.dim) conv_tokens<P, TAPS>(a, b, t0, tq, (is_k ? d.kv_heads * d.dim : 0) + kvh * d.dim + col, put);
        else for (int t = 0; t < 4; ++t) put(tq + t, zero);
    }
    __syncthreads();
    const float q_scale = rsqrtf(float(d.n_dim));
    #pragma unroll
    for (int t = warp; t < 2 * kDeltaBlock; t += 8) {             // unit vectors: 16 keys, then 16 queries
        float* row = (t < kDeltaBlock ? ks : qs - kDeltaBlock * ld) + t * ld;
        float ss = 0.f;
        for (int c = 4 * lane; c < R; c += 128) { const float4 v = load4<float>(row + c); ss += dot4(v, v); }
        const float f = rsqrtf(wave::dpp::reduce_sum(ss) + kUnitEps) * (t < kDeltaBlock ? 1.f : q_scale);
        for (int c = 4 * lane; c < R; c += 128) {
            const float4 v = load4<float>(row + c);
            store4<float>(row + c, make_float4(v.x * f, v.y * f, v.z * f, v.w * f));
        }
    }
    __syncthreads();
    if (!PLAIN) {
        // 120 dot products of keys with earlier ones, 136 of queries with keys: one per thread
        const bool of_q = tid >= 120;
        int n = of_q ? tid - 120 : tid, t = of_q ? 0 : 1;
        while (n >= t + of_q) { n -= t + of_q; ++t; }             // row t has t (keys) or t + 1 (queries) of them
        const float *r0 = (of_q ? qs : ks) + t * ld, *r1 = ks + n * ld;
        float s0 = 0.f, s1 = 0.f;
        for (int c = 0; c < R; c += 8) { s0 += dot4(load4<float>(r0 + c), load4<float>(r1 + c)); s1 += dot4(load4<float>(r0 + c + 4), load4<float>(r1 + c + 4)); }
        (of_q ? x.kq : x.kk)[n * 16 + t] = s0 + s1;
    }
    for (int h = kvh * d.group(); h < (kvh + 1) * d.group(); ++h) {
        if (tid < 2 * kDeltaBlock) {
            const int t = tid % 16;
            const float* ab = a.ab + (size_t(b) * a.Tn + t0 + t) * a.ld_ab;
            const bool live = t0 + t < a.Tn;                      // tokens past the call's leave S as it is
            if (tid < 16) x.g[t] = live ? decay(ab[h], a.a_log[h], a.dt_bias[h]) : 1.f;
            else          x.beta[t] = live ? step_size(ab[d.heads + h]) : 0.f;
        }
        __syncthreads();
        if (!PLAIN) {
            const int i = tid / 16, t = tid % 16;
            float r = 1.f;                                        // the decays between i and t
            for (int y = i + 1; y <= t; ++y) r *= x.g[y];
            x.l[t * 16 + i] = t > i ? x.beta[t] * r * x.kk[i * 16 + t] : 0.f;
            x.m[t * 16 + i] = t >= i ? r * x.kq[i * 16 + t] : 0.f;
            if (t == 15) x.tail[i] = r;
            if (i == 0) x.G[t] = r * x.g[0];
        }
        __syncthreads();
        if (!PLAIN && warp == 0) {
            // T = (1 + L)^-1 diag(beta): lane j solves column j, every row of L is read by all lanes
            const int j = lane % 16;
            float c[16];
            #pragma unroll
            for (int t = 0; t < 16; ++t) {
                float s = t == j ? x.beta[t] : 0.f;
                #pragma unroll
                for (int i4 = 0; i4 < t; i4 += 4) {
                    const float4 f = load4<float>(&x.l[t * 16 + i4]);
                    s -= f.x * c[i4];
                    if (i4 + 1 < t) s -= f.y * c[i4 + 1];
                    if (i4 + 2 < t) s -= f.z * c[i4 + 2];
                    if (i4 + 3 < t) s -= f.w * c[i4 + 3];
                }
                c[t] = s;
            }
            if (lane < 16) {
                const float G = x.G[j];
                #pragma unroll
                for (int t = 0; t < 16; ++t) { x.t_[j * 16 + t] = c[t]; x.tg[j * 16 + t] = c[t] * G; }
            }
        }
        for (int job = PLAIN ? tid : tid - 32; job >= 0 && job < d.vdim; job += PLAIN ? 256 : 224) {     // (columns, four tokens) of v
            const int col = 4 * (job % (d.vdim / 4)), tq = job / (d.vdim / 4) * 4;
            conv_tokens<P, TAPS>(a, b, t0, tq, 2 * d.kv_heads * d.dim + h * d.vdim + col, [&](int t, const float4& v) { store4<float>(vs + t * ldv + col, v); });
        }
        __syncthreads();
        if (!PLAIN) {
            const int j = tid / 16, t = tid % 16;
            float s = 0.f;
            #pragma unroll
            for (int i = 0; i < 16; ++i) s += x.m[t * 16 + i] * x.t_[j * 16 + i];
            x.mt[tid] = s; x.mtg[tid] = s * x.G[j];
            __syncthreads();
        }
        float* out = a.rows + ((size_t(b) * d.heads + h) * nblk + blk) * d.row_block(false);
        float* uo = a.cols + ((size_t(b) * d.heads + h) * (d.vdim / 16) * nblk + blk) * 512;        // slices of 16 columns, nblk * 512 apart
        if (PLAIN) {
            for (int e = tid; e < 8 * R; e += 256) {
                const int t = e / (R / 4), c = 4 * (e % (R / 4));
                store4<float>(out + e * 4, load4<float>((t < 16 ? ks + t * ld : qs + (t - 16) * ld) + c));
            }
            if (tid < 32) out[32 * R + tid] = tid < 16 ? x.g[tid] : x.beta[tid - 16];
            for (int e = tid; e < 4 * d.vdim; e += 256) {
                const int t = e / (d.vdim / 4), c = 4 * (e % (d.vdim / 4));
                store4<float>(uo + size_t(c / 16) * nblk * 512 + t * 16 + c % 16, load4<float>(vs + t * ldv + c));
            }
        } else {
            // two tokens t, four columns: sums over the block's tokens j with T and M T
            auto sums = [&](const float* rows, int ldr, int col, int t, const float* T, const float* MT, float4 (&st)[2], float4 (&sm)[2]) {
                st[0] = st[1] = sm[0] = sm[1] = zero;
                #pragma unroll
                for (int j = 0; j < 16; ++j) {
                    const float4 v = load4<float>(rows + j * ldr + col);
                    const float2 f = *reinterpret_cast<const float2*>(T + j * 16 + t), g = *reinterpret_cast<const float2*>(MT + j * 16 + t);
                    fma4(st[0], make_float4(f.x, f.x, f.x, f.x), v); fma4(st[1], make_float4(f.y, f.y, f.y, f.y), v);
                    fma4(sm[0], make_float4(g.x, g.x, g.x, g.x), v); fma4(sm[1], make_float4(g.y, g.y, g.y, g.y), v);
                }
            };
            for (int e = tid; e < 2 * R; e += 256) {
                const int col = 4 * (e % (R / 4)), t = 2 * (e / (R / 4));
                float4 st[2], sm[2];
                sums(ks, ld, col, t, x.tg, x.mtg, st, sm);
                #pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const float4 q = load4<float>(qs + (t + i) * ld + col), k = load4<float>(ks + (t + i) * ld + col);
                    const float G = x.G[t + i], f = x.tail[t + i];
                    store4<float>(out + (t + i) * R + col, st[i]);
                    store4<float>(out + (16 + t + i) * R + col, make_float4(G * q.x - sm[i].x, G * q.y - sm[i].y, G * q.z - sm[i].z, G * q.w - sm[i].w));
                    store4<float>(out + (32 + t + i) * R + col, make_float4(f * k.x, f * k.y, f * k.z, f * k.w));
                }
            }
            for (int e = tid; e < 2 * d.vdim; e += 256) {
                const int col = 4 * (e % (d.vdim / 4)), t = 2 * (e / (d.vdim / 4));
                float4 st[2], sm[2];
                sums(vs, ldv, col, t, x.t_, x.mt, st, sm);
                float* dst = uo + size_t(col / 16) * nblk * 512 + t * 16 + col % 16;
                #pragma unroll
                for (int i = 0; i < 2; ++i) { store4<float>(dst + i * 16, st[i]); store4<float>(dst + 256 + i * 16, sm[i]); }
            }
            if (tid < 4) out[48 * R + tid] = x.G[15];
        }
        __syncthreads();
    }
}

// ---- many tokens: the blocks ----------------------------------------------------------------------------------
constexpr int kBlockThreads = 128, kBlockStages = 3;
template <int DL, int NC> struct BlockSmem {                      // floats; DL rows of S per lane, NC columns
    static constexpr int R = 8 * DL, ROWS = 48 * R + 4, STAGE = ROWS + NC * 512;
    static constexpr int OFF_U = kBlockStages * STAGE, FLOATS = OFF_U + 4 * 64 * NC;         // per warp [16 t][4 NC columns]
    static constexpr int BYTES = FLOATS * 4 + 64;
};

template <int DL, int NC>
__global__ void __launch_bounds__(kBlockThreads) delta_blocks_kernel(const DeltaArgs a, int* sticky) {
    using Sh = BlockSmem<DL, NC>;
    constexpr int R = Sh::R, ST = kBlockStages, TT = 4 / NC;      // tokens whose sums are reduced together
    extern __shared__ __align__(128) float blk_smem[];
    uint64_t* full = reinterpret_cast<uint64_t*>(blk_smem + Sh::FLOATS);
    const DeltaDims& d = a.d;
    const int cta = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, grp = lane / 8, j = lane % 8;
    const int nblk = (a.Tn + kDeltaBlock - 1) / kDeltaBlock;
    const int slices = min(NC, d.vdim / 16 - cta * NC);           // 16-column slices of this CTA
    const float* src_rows = a.rows + (size_t(b) * d.heads + h) * nblk * Sh::ROWS;
    const float* src_cols = a.cols + ((size_t(b) * d.heads + h) * (d.vdim / 16) + cta * NC) * nblk * 512;
    if (threadIdx.x == 0) {
        for (int s = 0; s < ST; ++s) dme::mbar_init(&full[s], 1);
        dme::mbar_init_fence();
    }
    __syncthreads();
    auto fetch = [&](int n) {                                     // one thread: block n into its stage
        float* dst = blk_smem + (n % ST) * Sh::STAGE;
        dme::mbar_arrive_expect_tx(&full[n % ST], uint32_t(Sh::ROWS * 4 + slices * 2048));
        dme::copy_tile_1d(dst, src_rows + size_t(n) * Sh::ROWS, Sh::ROWS * 4, &full[n % ST]);
        for (int s = 0; s < slices; ++s) dme::copy_tile_1d(dst + Sh::ROWS + s * 512, src_cols + (size_t(s) * nblk + n) * 512, 2048, &full[n % ST]);
    };
    if (threadIdx.x == 0) for (int n = 0; n < ST && n < nblk; ++n) fetch(n);

    // S: columns col0 .. col0 + NC - 1, rows 32 x + 4 j .. + 3
    const int wcol = warp * 4 * NC, col0 = cta * 16 * NC + wcol + grp * NC;
    float* state = a.state + (size_t(b) * d.heads + h) * R * d.vdim;
    F2 S[NC][DL / 2];
    #pragma unroll
    for (int p = 0; p < DL / 2; ++p) {
        const int r = 32 * (p / 2) + 4 * j + 2 * (p % 2);
        #pragma unroll
        for (int c = 0; c < NC; ++c) {
            const bool live = a.pos0 > 0 && col0 + c < d.vdim;
            S[c][p] = live ? pair(state[size_t(r) * d.vdim + col0 + c], state[size_t(r + 1) * d.vdim + col0 + c]) : 0ull;
        }
    }
    // after the reduction a lane holds one sum: of the rows of u or of o, one of TT tokens, one of NC columns
    const bool of_o = (j & 4) != 0;
    const int my_t = (j & 3) / NC, my_c = grp * NC + (j & 3) % NC;                     // (column within the warp's)
    const int in_slice = (wcol + my_c) / 16 * 512 + (wcol + my_c) % 16;
    const bool live_out = cta * 16 * NC + wcol + my_c < d.vdim;
    float* o = a.o + size_t(b) * a.Tn * d.v_row() + size_t(h) * d.vdim + cta * 16 * NC + wcol + my_c;
    float* U = blk_smem + Sh::OFF_U + warp * 64 * NC;
    bool ok = true;
    for (int n = 0; n < nblk; ++n) {
        ok = dme::wait(&full[n % ST], uint32_t((n / ST) & 1), a.abort_word);
        // every warp is past block n - 1 here, so its stage can be filled again
        if (!__syncthreads_and(ok)) { ok = false; break; }
        if (threadIdx.x == 0 && n >= 1 && n - 1 + ST < nblk) fetch(n - 1 + ST);
        const float* st = blk_smem + (n % ST) * Sh::STAGE;
        const float* uo = st + Sh::ROWS + in_slice + (of_o ? 256 : 0);
        // ---- products with S --------------------------------------------------------------------------------------
        #pragma unroll 4
        for (int tg = 0; tg < kDeltaBlock / TT; ++tg) {
            const float base = uo[(tg * TT + my_t) * 16];
            F2 au[4], ao[4];
            #pragma unroll
            for (int y = 0; y < TT; ++y) {
                const float* wr = st + (tg * TT + y) * R + 4 * j;
                #pragma unroll
                for (int c = 0; c < NC; ++c) au[y * NC + c] = ao[y * NC + c] = 0ull;
                #pragma unroll
                for (int p = 0; p < DL / 4; ++p) {
                    const ulonglong2 wv = *reinterpret_cast<const ulonglong2*>(wr + 32 * p), qv = *reinterpret_cast<const ulonglong2*>(wr + 16 * R + 32 * p);
                    #pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        au[y * NC + c] = fma2(S[c][2 * p], wv.x, au[y * NC + c]); au[y * NC + c] = fma2(S[c][2 * p + 1], wv.y, au[y * NC + c]);
                        ao[y * NC + c] = fma2(S[c][2 * p], qv.x, ao[y * NC + c]); ao[y * NC + c] = fma2(S[c][2 * p + 1], qv.y, ao[y * NC + c]);
                    }
                }
            }
            float r4[4], r2[2];
            #pragma unroll
            for (int c = 0; c < 4; ++c) {
                const float su = sum2(au[c]), so = sum2(ao[c]);
                r4[c] = (of_o ? so : su) + __shfl_xor_sync(0xffffffffu, of_o ? su : so, 4);
            }
            #pragma unroll
            for (int c = 0; c < 2; ++c) r2[c] = ((j & 2) ? r4[2 + c] : r4[c]) + __shfl_xor_sync(0xffffffffu, (j & 2) ? r4[c] : r4[2 + c], 2);
            const float r1 = ((j & 1) ? r2[1] : r2[0]) + __shfl_xor_sync(0xffffffffu, (j & 1) ? r2[0] : r2[1], 1);
            const int t = tg * TT + my_t;
            if (!of_o) U[t * 4 * NC + my_c] = base - r1;
            else if (live_out && n * kDeltaBlock + t < a.Tn) o[size_t(n * kDeltaBlock + t) * d.v_row()] = base + r1;
        }
        __syncwarp();
        // ---- the update -------------------------------------------------------------------------------------------
        const float g = st[48 * R];
        const F2 g2 = pair(g, g);
        #pragma unroll
        for (int c = 0; c < NC; ++c)
            #pragma unroll
            for (int p = 0; p < DL / 2; ++p) S[c][p] = mul2(S[c][p], g2);
        #pragma unroll(NC == 1 ? 16 : 8)
        for (int t = 0; t < kDeltaBlock; ++t) {
            F2 u[NC];
            if constexpr (NC == 4) {
                const float4 v = load4<float>(U + t * 16 + grp * 4);
                u[0] = pair(v.x, v.x); u[1] = pair(v.y, v.y); u[2] = pair(v.z, v.z); u[3] = pair(v.w, v.w);
            } else if constexpr (NC == 2) {
                const float2 v = *reinterpret_cast<const float2*>(U + t * 8 + grp * 2);
                u[0] = pair(v.x, v.x); u[1] = pair(v.y, v.y);
            } else { const float v = U[t * 4 + grp]; u[0] = pair(v, v); }
            #pragma unroll
            for (int p = 0; p < DL / 4; ++p) {
                const ulonglong2 kv = *reinterpret_cast<const ulonglong2*>(st + (32 + t) * R + 32 * p + 4 * j);
                #pragma unroll
                for (int c = 0; c < NC; ++c) { S[c][2 * p] = fma2(kv.x, u[c], S[c][2 * p]); S[c][2 * p + 1] = fma2(kv.y, u[c], S[c][2 * p + 1]); }
            }
        }
        __syncwarp();                                             // U is read before the next block writes it
    }
    if (!ok) { if (threadIdx.x == 0) { atomicExch(a.abort_word, 1); atomicExch(sticky, 1); } return; }
    #pragma unroll
    for (int p = 0; p < DL / 2; ++p) {
        const int r = 32 * (p / 2) + 4 * j + 2 * (p % 2);
        #pragma unroll
        for (int c = 0; c < NC; ++c)
            if (col0 + c < d.vdim) {
                const float2 v = unpair(S[c][p]);
                state[size_t(r) * d.vdim + col0 + c] = v.x; state[size_t(r + 1) * d.vdim + col0 + c] = v.y;
            }
    }
}

// ---- many tokens on the tensor cores (16-bit sessions) ----------------------------------------------------------
// The same two kernels with their products as mma_fp32.  Rows of k and q (and of the block form's first two matrices)
// are 64 bytes longer than S's: a quarter-warp's 16-byte reads of two rows fall on different banks.
constexpr int kMatLd = 20;              // floats between the rows of a 16 x 16 matrix: 16-byte reads of eight rows on different banks
struct PrepMma {
    float kk[16 * kMatLd], kq[16 * kMatLd];        // (k_i.k_t), (k_i.q_t) at [t][i], before the unit lengths
    float l[16 * kMatLd], m[16 * kMatLd];          // the triangles of u and o at [t][i]
    float t_[256];                                 // T at [j][t]
    float coef[4][16 * kMatLd];                    // [t][j]: T, M T, and both times G_j / |k_j|
    float g[16], beta[16], G[16], tail[16], rk[16], rq[16];
};

template <typename P, int TAPS, int X>
__global__ void __launch_bounds__(256, 3) delta_prepare_mma_kernel(const DeltaArgs a) {
    extern __shared__ __align__(16) float prep_smem[];
    __shared__ __align__(16) PrepMma x;
    constexpr int R = 16 * X, ld = R + 16;
    const DeltaDims& d = a.d;
    const int ldv = d.vdim + 8;
    float *ks = prep_smem, *qs = ks + kDeltaBlock * ld, *vs = qs + kDeltaBlock * ld;
    const int blk = blockIdx.x, nblk = gridDim.x, kvh = blockIdx.y, b = blockIdx.z, t0 = blk * kDeltaBlock;
    const int tid = threadIdx.x, warp = tid / 32, lane = tid % 32, r = lane / 4, q = lane % 4;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int col = 4 * lane; col < R; col += 128) {               // a warp: q or k, four tokens
        const int tq = warp % 4 * 4;
        float* dst = (warp >= 4 ? ks : qs) + col;
        auto put = [&](int t, const float4& v) { store4<float>(dst + t * ld, v); };
        if (col < d.dim) conv_tokens<P, TAPS, true>(a, b, t0, tq, (warp >= 4 ? d.kv_heads * d.dim : 0) + kvh * d.dim + col, put);
        else for (int t = 0; t < 4; ++t) put(tq + t, zero);
    }
    __syncthreads();
    if (warp < 4) {
        // dot products: warp (kind, eight keys i); rows t.  A k-step's lane q takes columns 16 y + 4 q + {0, 1} or {2, 3}
        const bool of_q = warp >= 2;
        const int i0 = (warp & 1) * 8;
        const float *ra = (of_q ? qs : ks) + r * ld + 4 * q, *rb = ks + (i0 + r) * ld + 4 * q;
        float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        #pragma unroll
        for (int c = 0; c < R; c += 16) {
            const float4 a0 = load4<float>(ra + c), a1 = load4<float>(ra + 8 * ld + c), bv = load4<float>(rb + c);
            const Split s0[4] = {split(a0.x), split(a1.x), split(a0.y), split(a1.y)}, s1[4] = {split(a0.z), split(a1.z), split(a0.w), split(a1.w)};
            mma_fp32(acc[0], s0, split(bv.x), split(bv.y));
            mma_fp32(acc[1], s1, split(bv.z), split(bv.w));
        }
        float* dots = of_q ? x.kq : x.kk;
        #pragma unroll
        for (int e = 0; e < 4; ++e) dots[(r + 8 * (e >> 1)) * kMatLd + i0 + 2 * q + (e & 1)] = acc[0][e] + acc[1][e];
    } else {
        const float q_scale = rsqrtf(float(d.n_dim));
        float ss[8];                                              // unit lengths: warps 4, 5 the keys, 6, 7 the queries
        const float* row = (warp < 6 ? ks : qs) + (warp & 1) * 8 * ld;
        #pragma unroll
        for (int t = 0; t < 8; ++t) {
            ss[t] = 0.f;
            for (int c = 4 * lane; c < R; c += 128) { const float4 v = load4<float>(row + t * ld + c); ss[t] += dot4(v, v); }
        }
        #pragma unroll
        for (int t = 0; t < 8; ++t) {
            const float f = rsqrtf(wave::dpp::reduce_sum(ss[t]) + kUnitEps);
            if (lane == 0) (warp < 6 ? x.rk : x.rq)[(warp & 1) * 8 + t] = warp < 6 ? f : f * q_scale;
        }
    }
    for (int h = kvh * d.group(); h < (kvh + 1) * d.group(); ++h) {
        if (tid >= 224) {
            const int t = tid % 16;
            const float* ab = a.ab + (size_t(b) * a.Tn + t0 + t) * a.ld_ab;
            const bool live = t0 + t < a.Tn;                      // tokens past the call's leave S as it is
            if (tid < 240) x.g[t] = live ? decay(ab[h], a.a_log[h], a.dt_bias[h]) : 1.f;
            else           x.beta[t] = live ? step_size(ab[d.heads + h]) : 0.f;
        }
        __syncthreads();
        {
            const int i = tid / 16, t = tid % 16;
            float f = t > i ? x.g[t] : 1.f;                       // the decays between i and t: a running product over the 16 lanes
            #pragma unroll
            for (int y = 1; y < 16; y *= 2) { const float o = __shfl_up_sync(0xffffffffu, f, y, 16); if (t >= y) f *= o; }
            x.l[t * kMatLd + i] = t > i ? x.beta[t] * f * x.kk[t * kMatLd + i] * x.rk[i] * x.rk[t] : 0.f;
            x.m[t * kMatLd + i] = t >= i ? f * x.kq[t * kMatLd + i] * x.rk[i] * x.rq[t] : 0.f;
            if (t == 15) x.tail[i] = f * x.rk[i];
            if (i == 0) x.G[t] = f * x.g[0];
        }
        __syncthreads();
        float* out = a.rows + ((size_t(b) * d.heads + h) * nblk + blk) * d.row_block(true);
        if (warp == 0) {
            // T = (1 + L)^-1 diag(beta): lane j solves column j, every row of L is read by all lanes
            const int j = lane % 16;
            float c[16];
            #pragma unroll
            for (int t = 0; t < 16; ++t) {
                float s = t == j ? x.beta[t] : 0.f;
                #pragma unroll
                for (int i4 = 0; i4 < t; i4 += 4) {
                    const float4 f = load4<float>(&x.l[t * kMatLd + i4]);
                    s -= f.x * c[i4];
                    if (i4 + 1 < t) s -= f.y * c[i4 + 1];
                    if (i4 + 2 < t) s -= f.z * c[i4 + 2];
                    if (i4 + 3 < t) s -= f.w * c[i4 + 3];
                }
                c[t] = s;
            }
            if (lane < 16) {
                #pragma unroll
                for (int t = 0; t < 16; t += 4) store4<float>(&x.t_[j * 16 + t], make_float4(c[t], c[t + 1], c[t + 2], c[t + 3]));
            }
        } else if (warp < 4) {
            const int t = lane % 4 * 4;                           // the update's keys, [row][16 t]
            const float f0 = x.tail[t], f1 = x.tail[t + 1], f2 = x.tail[t + 2], f3 = x.tail[t + 3];
            for (int c = (warp - 1) * 8 + r; c < R; c += 24) {
                const float* k = ks + t * ld + c;
                store4<float>(out + 32 * ld + c * 16 + t, make_float4(k[0] * f0, k[ld] * f1, k[2 * ld] * f2, k[3 * ld] * f3));
            }
            if (tid < 36) out[32 * ld + 16 * R + tid - 32] = x.G[15];
        } else {
            for (int col = 4 * lane; col < d.vdim; col += 128)    // v, four tokens a warp
                conv_tokens<P, TAPS, true>(a, b, t0, (warp - 4) * 4, 2 * d.kv_heads * d.dim + h * d.vdim + col, [&](int t, const float4& v) { store4<float>(vs + t * ldv + col, v); });
        }
        __syncthreads();
        {
            const int j = tid / 16, t = tid % 16;
            float s = 0.f;
            #pragma unroll
            for (int i = 0; i < 16; i += 4) s += dot4(load4<float>(&x.m[t * kMatLd + i]), load4<float>(&x.t_[j * 16 + i]));
            const float f = x.G[j] * x.rk[j], T = x.t_[tid];
            x.coef[0][t * kMatLd + j] = T; x.coef[1][t * kMatLd + j] = s;
            x.coef[2][t * kMatLd + j] = T * f; x.coef[3][t * kMatLd + j] = s * f;
        }
        __syncthreads();
        // A fragments of two of the 16 x 16 matrices: k-steps j = q, q + 4 and q + 8, q + 12
        Split f0[2][4], f1[2][4];
        auto take = [&](int which) {
            #pragma unroll
            for (int y = 0; y < 2; ++y)
                #pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int at = (r + 8 * (e & 1)) * kMatLd + 8 * y + q + 4 * (e >> 1);
                    f0[y][e] = split(x.coef[which][at]); f1[y][e] = split(x.coef[which + 1][at]);
                }
        };
        auto sums = [&](const float* col, int ldr, float (&s0)[4], float (&s1)[4]) {        // over the block's tokens, eight columns
            #pragma unroll
            for (int e = 0; e < 4; ++e) s0[e] = s1[e] = 0.f;
            #pragma unroll
            for (int y = 0; y < 2; ++y) {
                const Split b0 = split(col[(8 * y + q) * ldr + r]), b1 = split(col[(8 * y + q + 4) * ldr + r]);
                mma_fp32(s0, f0[y], b0, b1);
                mma_fp32(s1, f1[y], b0, b1);
            }
        };
        take(2);
        #pragma unroll
        for (int n0 = 0; n0 < R / 8; n0 += 8) {
            const int n = n0 + warp;
            if (n >= R / 8) break;
            float w[4], s[4];
            sums(ks + 8 * n, ld, w, s);
            #pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = r + 8 * e, c = 8 * n + 2 * q;
                const float2 qv = *reinterpret_cast<const float2*>(qs + t * ld + c);
                const float f = x.G[t] * x.rq[t];
                *reinterpret_cast<float2*>(out + t * ld + c) = make_float2(w[2 * e], w[2 * e + 1]);
                *reinterpret_cast<float2*>(out + (16 + t) * ld + c) = make_float2(f * qv.x - s[2 * e], f * qv.y - s[2 * e + 1]);
            }
        }
        take(0);
        float* uo = a.cols + ((size_t(b) * d.heads + h) * (d.vdim / 16) * nblk + blk) * 512;        // slices of 16 columns [u, o][16][16 t], nblk * 512 apart
        for (int n = warp; n < d.vdim / 8; n += 8) {
            float u[4], o[4];
            sums(vs + 8 * n, ldv, u, o);
            float* dst = uo + size_t(n / 2) * nblk * 512 + (n % 2 * 8 + 2 * q) * 16 + r;
            #pragma unroll
            for (int e = 0; e < 4; ++e) { dst[(e & 1) * 16 + 8 * (e >> 1)] = u[e]; dst[256 + (e & 1) * 16 + 8 * (e >> 1)] = o[e]; }
        }
        __syncthreads();
    }
}

// A group of KS warps owns 16 columns of S, each of them a KS-th of the rows.  Everything is computed transposed: S^T lies in
// accumulator fragments (columns x rows), which are operand fragments as they are when the k index runs over rows in the
// order the accumulators hold them -- tile 2 y + z of a lane q: rows 16 y + 4 q + 2 z + {0, 1} -- and u^T, an accumulator, is an
// operand of the update the same way (tokens 4 q + 2 z + {0, 1}).  The warps of a group add up their partial products
// through shared memory; nothing else crosses lanes.
template <int X> struct BlockMmaSmem {                            // floats; X groups of 16 rows of S
    static constexpr int R = 16 * X, LD = R + 16, ROWS = 32 * LD + 16 * R + 4;
    static constexpr int stage(int slices) { return ROWS + slices * 512; }
    static constexpr int bytes(int slices, int ks) { return (kBlockStages * stage(slices) + (ks > 1 ? 2 * slices * ks * 512 : 0)) * 4 + 64; }
};

template <int X, int KS>
__global__ void __launch_bounds__(kBlockThreads) delta_blocks_mma_kernel(const DeltaArgs a, int* sticky) {
    using Sh = BlockMmaSmem<X>;
    constexpr int R = Sh::R, LD = Sh::LD, ST = kBlockStages, XW = X / KS;
    static_assert(X % KS == 0, "whole row groups per warp");
    extern __shared__ __align__(128) float blk_smem[];
    const int group = blockDim.x / (32 * KS), stage = Sh::stage(group);      // slices of 16 columns per CTA
    float* xch = blk_smem + ST * stage;                           // [block's parity][slice][part][4][32 lanes][4]
    uint64_t* full = reinterpret_cast<uint64_t*>(xch + (KS > 1 ? 2 * group * KS * 512 : 0));
    const DeltaDims& d = a.d;
    const int h = blockIdx.y, b = blockIdx.z;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, r = lane / 4, q = lane % 4, part = warp % KS, sl = warp / KS;
    const int nblk = (a.Tn + kDeltaBlock - 1) / kDeltaBlock;
    const int slice0 = blockIdx.x * group, slices = min(group, d.vdim / 16 - slice0);
    const bool mine = sl < slices;
    const float* src_rows = a.rows + (size_t(b) * d.heads + h) * nblk * Sh::ROWS;
    const float* src_cols = a.cols + ((size_t(b) * d.heads + h) * (d.vdim / 16) + slice0) * nblk * 512;
    if (threadIdx.x == 0) {
        for (int s = 0; s < ST; ++s) dme::mbar_init(&full[s], 1);
        dme::mbar_init_fence();
    }
    __syncthreads();
    auto fetch = [&](int n) {                                     // one thread: block n into its stage
        float* dst = blk_smem + (n % ST) * stage;
        dme::mbar_arrive_expect_tx(&full[n % ST], uint32_t(Sh::ROWS * 4 + slices * 2048));
        dme::copy_tile_1d(dst, src_rows + size_t(n) * Sh::ROWS, Sh::ROWS * 4, &full[n % ST]);
        for (int s = 0; s < slices; ++s) dme::copy_tile_1d(dst + Sh::ROWS + s * 512, src_cols + (size_t(s) * nblk + n) * 512, 2048, &full[n % ST]);
    };
    if (threadIdx.x == 0) for (int n = 0; n < ST && n < nblk; ++n) fetch(n);

    const int col = (slice0 + sl) * 16 + r, y0 = part * XW;       // and col + 8
    float* state = a.state + (size_t(b) * d.heads + h) * R * d.vdim + col;
    auto row_of = [&](int y, int z, int e) { return size_t(16 * (y0 + y) + 4 * q + 2 * z + e) * d.vdim; };
    float S[XW][2][4];
    #pragma unroll
    for (int y = 0; y < XW; ++y)
        #pragma unroll
        for (int z = 0; z < 2; ++z)
            #pragma unroll
            for (int e = 0; e < 4; ++e) S[y][z][e] = mine && a.pos0 > 0 ? state[row_of(y, z, e & 1) + 8 * (e >> 1)] : 0.f;
    float* o = a.o + size_t(b) * a.Tn * d.v_row() + size_t(h) * d.vdim + col;
    const int n_tok = 4 * (r / 2) + r % 2;                        // the token (and row) that column r of an operand tile stands for, z = 0
    bool ok = true;
    for (int n = 0; n < nblk; ++n) {
        ok = dme::wait(&full[n % ST], uint32_t((n / ST) & 1), a.abort_word);
        // All warps meet once a block, here or, where partial products are exchanged, there: by then every one of them is past
        // block n - 1, whose stage can be filled again.
        auto meet = [&] {
            ok = __syncthreads_and(ok);
            if (ok && threadIdx.x == 0 && n >= 1 && n - 1 + ST < nblk) fetch(n - 1 + ST);
            return ok;
        };
        if (KS == 1) {
            if (!meet()) break;
            if (!mine) continue;
        }
        const float* st = blk_smem + (n % ST) * stage;
        // ---- products with S: [u, tokens z = 0, 1; o, tokens z = 0, 1].  The passes of the four are interleaved: four chains ------
        float acc[4][4];
        #pragma unroll
        for (int k = 0; k < 4; ++k) acc[k][0] = acc[k][1] = acc[k][2] = acc[k][3] = 0.f;
        #pragma unroll
        for (int y = 0; y < XW; ++y) {
            Split f[4][4];
            #pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float4 v = load4<float>(st + (16 * (k >> 1) + n_tok + 2 * (k & 1)) * LD + 16 * (y0 + y) + 4 * q);
                f[k][0] = split(v.x); f[k][1] = split(v.y); f[k][2] = split(v.z); f[k][3] = split(v.w);
            }
            #pragma unroll
            for (int z = 0; z < 2; ++z) {
                const float (&c)[4] = S[y][z];
                const Split s[4] = {split(c[0]), split(c[2]), split(c[1]), split(c[3])};
                #pragma unroll
                for (int k = 0; k < 4; ++k) mma_tf32(acc[k], s[0].lo, s[1].lo, s[2].lo, s[3].lo, f[k][2 * z].hi, f[k][2 * z + 1].hi);
                #pragma unroll
                for (int k = 0; k < 4; ++k) mma_tf32(acc[k], s[0].hi, s[1].hi, s[2].hi, s[3].hi, f[k][2 * z].lo, f[k][2 * z + 1].lo);
                #pragma unroll
                for (int k = 0; k < 4; ++k) mma_tf32(acc[k], s[0].hi, s[1].hi, s[2].hi, s[3].hi, f[k][2 * z].hi, f[k][2 * z + 1].hi);
            }
        }
        if constexpr (KS > 1) {
            float* x = xch + ((n & 1) * group + sl) * KS * 512;
            #pragma unroll
            for (int k = 0; k < 4; ++k) store4<float>(x + part * 512 + k * 128 + lane * 4, make_float4(acc[k][0], acc[k][1], acc[k][2], acc[k][3]));
            if (!meet()) break;
            if (!mine) continue;
            #pragma unroll
            for (int k = 0; k < 2; ++k) {                         // u, in the same order in every warp
                float4 v = load4<float>(x + k * 128 + lane * 4);
                #pragma unroll
                for (int p = 1; p < KS; ++p) { const float4 y = load4<float>(x + p * 512 + k * 128 + lane * 4); v.x += y.x; v.y += y.y; v.z += y.z; v.w += y.w; }
                acc[k][0] = v.x; acc[k][1] = v.y; acc[k][2] = v.z; acc[k][3] = v.w;
            }
        }
        const float* uo = st + Sh::ROWS + sl * 512 + r * 16 + 4 * q;
        Split u[2][4];                                            // operand fragments of u^T
        #pragma unroll
        for (int c = 0; c < 2; ++c) {                             // columns col, col + 8
            const float4 u0 = load4<float>(uo + c * 128);
            u[0][c] = split(u0.x - acc[0][2 * c]); u[0][2 + c] = split(u0.y - acc[0][2 * c + 1]);
            u[1][c] = split(u0.z - acc[1][2 * c]); u[1][2 + c] = split(u0.w - acc[1][2 * c + 1]);
        }
        #pragma unroll
        for (int e = 0; e < 4 / KS; ++e) {                        // o: the group's warps share (column half, tokens z)
            const int job = KS == 1 ? e : part * (4 / KS) + e, c = job >> 1, z = job & 1;
            float2 v = *reinterpret_cast<const float2*>(uo + 256 + c * 128 + 2 * z);
            if constexpr (KS == 1) { v.x += acc[2 + z][2 * c]; v.y += acc[2 + z][2 * c + 1]; }
            else {
                #pragma unroll
                for (int p = 0; p < KS; ++p) {
                    const float2 y = *reinterpret_cast<const float2*>(xch + (((n & 1) * group + sl) * KS + p) * 512 + (2 + z) * 128 + lane * 4 + 2 * c);
                    v.x += y.x; v.y += y.y;
                }
            }
            const int t = n * kDeltaBlock + 4 * q + 2 * z;
            if (t < a.Tn) o[size_t(t) * d.v_row() + 8 * c] = v.x;
            if (t + 1 < a.Tn) o[size_t(t + 1) * d.v_row() + 8 * c] = v.y;
        }
        // ---- the update, two tiles at a time -----------------------------------------------------------------------------------
        const float g = st[32 * LD + 16 * R];
        #pragma unroll
        for (int y = 0; y < XW; ++y) {
            Split f[2][4];
            #pragma unroll
            for (int z = 0; z < 2; ++z) {
                const float4 v = load4<float>(st + 32 * LD + (16 * (y0 + y) + n_tok + 2 * z) * 16 + 4 * q);
                f[z][0] = split(v.x); f[z][1] = split(v.y); f[z][2] = split(v.z); f[z][3] = split(v.w);
                #pragma unroll
                for (int e = 0; e < 4; ++e) S[y][z][e] *= g;
            }
            #pragma unroll
            for (int t = 0; t < 2; ++t) {
                #pragma unroll
                for (int z = 0; z < 2; ++z) mma_tf32(S[y][z], u[t][0].lo, u[t][1].lo, u[t][2].lo, u[t][3].lo, f[z][2 * t].hi, f[z][2 * t + 1].hi);
                #pragma unroll
                for (int z = 0; z < 2; ++z) mma_tf32(S[y][z], u[t][0].hi, u[t][1].hi, u[t][2].hi, u[t][3].hi, f[z][2 * t].lo, f[z][2 * t + 1].lo);
                #pragma unroll
                for (int z = 0; z < 2; ++z) mma_tf32(S[y][z], u[t][0].hi, u[t][1].hi, u[t][2].hi, u[t][3].hi, f[z][2 * t].hi, f[z][2 * t + 1].hi);
            }
        }
    }
    if (!ok) { if (threadIdx.x == 0) { atomicExch(a.abort_word, 1); atomicExch(sticky, 1); } return; }
    if (!mine) return;
    #pragma unroll
    for (int y = 0; y < XW; ++y)
        #pragma unroll
        for (int z = 0; z < 2; ++z)
            #pragma unroll
            for (int e = 0; e < 4; ++e) state[row_of(y, z, e & 1) + 8 * (e >> 1)] = S[y][z][e];
}

// Token by token, any size: one warp per column of S, rows lane, lane + 32, ...
template <int NR>
__global__ void __launch_bounds__(256) delta_plain_kernel(const DeltaArgs a) {
    const DeltaDims& d = a.d;
    const int R = d.rows(), warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int col = blockIdx.x * 8 + warp, h = blockIdx.y, b = blockIdx.z;
    if (col >= d.vdim) return;
    const int nblk = (a.Tn + kDeltaBlock - 1) / kDeltaBlock;
    const float* rows = a.rows + (size_t(b) * d.heads + h) * nblk * d.row_block(false);
    const float* v = a.cols + ((size_t(b) * d.heads + h) * (d.vdim / 16) + col / 16) * nblk * 512 + col % 16;
    float* state = a.state + (size_t(b) * d.heads + h) * R * d.vdim + col;
    float S[NR];
    #pragma unroll
    for (int i = 0; i < NR; ++i) { const int r = lane + 32 * i; S[i] = a.pos0 > 0 && r < R ? state[size_t(r) * d.vdim] : 0.f; }
    for (int t = 0; t < a.Tn; ++t) {
        const int n = t / kDeltaBlock, x = t % kDeltaBlock;
        const float* blk = rows + size_t(n) * d.row_block(false);
        const float *k = blk + x * R, *q = blk + (16 + x) * R;
        const float g = blk[32 * R + x], beta = blk[32 * R + 16 + x];
        float kr[NR], p = 0.f, o = 0.f;
        #pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int r = lane + 32 * i;
            kr[i] = r < R ? k[r] : 0.f;
            S[i] *= g;
            p += S[i] * kr[i];
        }
        const float u = beta * (v[size_t(n) * 512 + x * 16] - wave::dpp::reduce_sum(p));
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

// ---- many tokens: norm and gate -----------------------------------------------------------------------------------
// W lanes per (token, head), eight columns a lane and CH of them; further CTAs keep the convolutions' last inputs, a quad
// of channels per thread.
template <typename T, typename P, int W, int CH>
__global__ void __launch_bounds__(256) delta_finish_kernel(const DeltaArgs a, unsigned rows, unsigned norm_ctas) {
    const DeltaDims& d = a.d;
    if (blockIdx.x >= norm_ctas) {
        const int keep = min(d.taps, a.Tn), quads = d.channels() / 4;
        const size_t i = size_t(blockIdx.x - norm_ctas) * 256 + threadIdx.x;
        if (i >= size_t(a.batch) * keep * quads) return;
        const int c = 4 * int(i % quads), b = int(i / quads / keep), t = a.Tn - 1 - int(i / quads % keep);
        store4<float>(a.ring + (size_t(b) * d.taps + (a.pos0 + t) % d.taps) * d.channels() + c, conv_input<P>(a, b, t, c));
        return;
    }
    const unsigned u = (blockIdx.x * 256u + threadIdx.x) / W, r = u < rows ? u : rows - 1;        // [token][head], vdim columns each
    const int c0 = threadIdx.x % W * 8;
    const unsigned tok = r / unsigned(d.heads);
    const P* gate = static_cast<const P*>(a.proj) + size_t(tok) * a.ldp + d.g_col() + (r - tok * d.heads) * d.vdim;
    const float* o = a.o + size_t(r) * d.vdim;
    float v[CH][8], s[CH][8];
    float ss = 0.f;
    #pragma unroll
    for (int i = 0; i < CH; ++i) {
        const int c = c0 + 8 * W * i;
        if (c < d.vdim) {
            load8<float>(o + c, v[i]);
            load8<P>(gate + c, s[i]);
            #pragma unroll
            for (int k = 0; k < 8; ++k) ss += v[i][k] * v[i][k];
        }
    }
    const float f = rsqrtf(wave::lane_group_reduce<W>(ss, wave::SumOp{}) / d.n_vdim + a.eps);
    if (u >= rows) return;
    #pragma unroll
    for (int i = 0; i < CH; ++i) {
        const int c = c0 + 8 * W * i;
        if (c >= d.vdim) continue;
        float w[8];
        load8<float>(a.norm + c, w);
        #pragma unroll
        for (int k = 0; k < 8; ++k) v[i][k] *= f * w[k] * silu<!std::is_same_v<T, float>>(s[i][k]);
        store8<T>(static_cast<T*>(a.out) + size_t(r) * d.vdim + c, v[i]);
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

template <int DL, int NC>
int launch_blocks_nc(const DeltaArgs& a, cudaStream_t st) {
    using Sh = BlockSmem<DL, NC>;
    int* sticky = device_status_ptr();
    if (!sticky) return B200P_E_NO_DEVICE;
    auto kern = delta_blocks_kernel<DL, NC>;
    if (cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::BYTES)) return int(e);
    kern<<<dim3(unsigned((a.d.vdim / 16 + NC - 1) / NC), unsigned(a.d.heads), unsigned(a.batch)), kBlockThreads, Sh::BYTES, st>>>(a, sticky);
    return launched();
}
// More columns per lane read less shared memory per FMA, fewer make more warps: as many as leave every scheduler one.
template <int DL>
int launch_blocks(const DeltaArgs& a, cudaStream_t st) {
    const long long warps = (long long)a.batch * a.d.heads * (a.d.vdim / 4), want = 4LL * (sm_count() > 0 ? sm_count() : 148);      // with NC = 1
    const int forced = tuning(KNOB_DELTA_COLUMNS, 0);
    const int nc = forced > 0 ? forced : warps >= 4 * want ? 4 : warps >= 2 * want ? 2 : 1;
    return nc >= 4 ? launch_blocks_nc<DL, 4>(a, st) : nc >= 2 ? launch_blocks_nc<DL, 2>(a, st) : launch_blocks_nc<DL, 1>(a, st);
}

template <int X, int KS>
int launch_blocks_mma_ks(const DeltaArgs& a, int group, cudaStream_t st) {
    using Sh = BlockMmaSmem<X>;
    int* sticky = device_status_ptr();
    if (!sticky) return B200P_E_NO_DEVICE;
    auto kern = delta_blocks_mma_kernel<X, KS>;
    if (cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::bytes(kBlockThreads / 32 / KS, KS))) return int(e);
    kern<<<dim3(unsigned((a.d.vdim / 16 + group - 1) / group), unsigned(a.d.heads), unsigned(a.batch)), 32 * KS * group, Sh::bytes(group, KS), st>>>(a, sticky);
    return launched();
}
// Few columns in all: several warps share a slice's rows, so that every scheduler has one; many: a warp takes all rows and
// four slices share a CTA's copies.
template <int X>
int launch_blocks_mma(const DeltaArgs& a, cudaStream_t st) {
    const long long slices = (long long)a.batch * a.d.heads * (a.d.vdim / 16), sms = sm_count() > 0 ? sm_count() : 148;
    const int forced = tuning(KNOB_DELTA_COLUMNS, 0);
    const int ks = forced == 1 ? 4 : forced == 2 ? 2 : forced >= 4 ? 1 : slices <= 2 * sms ? 4 : slices <= 3 * sms ? 2 : 1;
    if constexpr (X % 4 == 0) { if (ks == 4) return launch_blocks_mma_ks<X, 4>(a, 1, st); }
    if (ks >= 2) return launch_blocks_mma_ks<X, 2>(a, slices <= sms ? 1 : 2, st);
    return launch_blocks_mma_ks<X, 1>(a, 4, st);
}

template <typename P, int X>
int launch_prepare_mma_x(const DeltaArgs& a, int nblk, cudaStream_t st) {
    const size_t smem = size_t(kDeltaBlock) * (2 * (16 * X + 16) + a.d.vdim + 8) * 4;
    auto kern = a.d.taps == 4 ? delta_prepare_mma_kernel<P, 4, X> : delta_prepare_mma_kernel<P, 0, X>;
    if (smem > 36 * 1024)
        if (cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem))) return int(e);
    kern<<<dim3(unsigned(nblk), unsigned(a.d.kv_heads), unsigned(a.batch)), 256, smem, st>>>(a);
    return launched();
}
// (16-bit sessions: the projection has their type when there are many tokens)
int launch_prepare_mma(const DeltaArgs& a, int nblk, cudaStream_t st) {
    switch (a.d.rows() / 32) {
        case 1: return launch_prepare_mma_x<T16, 2>(a, nblk, st);
        case 2: return launch_prepare_mma_x<T16, 4>(a, nblk, st);
        case 3: return launch_prepare_mma_x<T16, 6>(a, nblk, st);
    }
    return launch_prepare_mma_x<T16, 8>(a, nblk, st);
}

template <typename T, typename P>
int launch_finish(const DeltaArgs& a, cudaStream_t st) {
    const DeltaDims& d = a.d;
    const unsigned rows = unsigned(a.batch) * a.Tn * d.heads;
    const size_t tail = size_t(a.batch) * (d.taps < a.Tn ? d.taps : a.Tn) * (d.channels() / 4);
    auto run = [&](auto kern, unsigned W) {
        const unsigned ctas = (rows + 256 / W - 1) / (256 / W);
        kern<<<ctas + unsigned((tail + 255) / 256), 256, 0, st>>>(a, rows, ctas);
        return launched();
    };
    const int lanes = d.vdim / 8;
    if (lanes <= 2) return run(delta_finish_kernel<T, P, 2, 1>, 2);
    if (lanes <= 4) return run(delta_finish_kernel<T, P, 4, 1>, 4);
    if (lanes <= 8) return run(delta_finish_kernel<T, P, 8, 1>, 8);
    if (lanes <= 16) return run(delta_finish_kernel<T, P, 16, 1>, 16);
    return run(delta_finish_kernel<T, P, 32, 2>, 32);
}

template <typename P, bool PLAIN>
int launch_prepare(const DeltaArgs& a, int nblk, cudaStream_t st) {
    const size_t smem = size_t(kDeltaBlock) * (2 * (a.d.rows() + 4) + a.d.vdim + 4) * 4;
    auto kern = a.d.taps == 4 ? delta_prepare_kernel<P, 4, PLAIN> : delta_prepare_kernel<P, 0, PLAIN>;
    if (smem > 36 * 1024)
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
    if (d.rows() > 512 || d.vdim > 512) return B200P_E_DIM;
    if (d.heads > 65535 || a.batch > 65535 || (long long)a.batch * a.Tn * d.heads * 32 > 0xffffffffLL) return B200P_E_RANGE;
    const bool f32 = a.proj_dtype == B200P_F32, plain = d.rows() > 128 || tuning(KNOB_DELTA_PLAIN, 0) != 0;
    const int nblk = (a.Tn + kDeltaBlock - 1) / kDeltaBlock;
    // fp32 sessions stay off the tensor cores
    const bool tensor = !plain && a.dtype != B200P_F32 && !f32 && tuning(KNOB_DELTA_TENSOR, 1) != 0;
    int rc = tensor ? launch_prepare_mma(a, nblk, st)
           : f32 ? (plain ? launch_prepare<float, true>(a, nblk, st) : launch_prepare<float, false>(a, nblk, st))
                 : (plain ? launch_prepare<T16, true>(a, nblk, st) : launch_prepare<T16, false>(a, nblk, st));
    if (rc) return rc;
    if (tensor) {
        rc = d.rows() <= 32 ? launch_blocks_mma<2>(a, st) : d.rows() <= 64 ? launch_blocks_mma<4>(a, st) : d.rows() <= 96 ? launch_blocks_mma<6>(a, st) : launch_blocks_mma<8>(a, st);
    } else if (!plain) {
        rc = d.rows() <= 32 ? launch_blocks<4>(a, st) : d.rows() <= 64 ? launch_blocks<8>(a, st) : d.rows() <= 96 ? launch_blocks<12>(a, st) : launch_blocks<16>(a, st);
    } else {
        const dim3 grid(unsigned((d.vdim + 7) / 8), unsigned(d.heads), unsigned(a.batch));
        if (d.rows() <= 128) delta_plain_kernel<4><<<grid, 256, 0, st>>>(a);
        else delta_plain_kernel<16><<<grid, 256, 0, st>>>(a);
        rc = launched();
    }
    if (rc) return rc;
    return a.dtype == B200P_F32 ? launch_finish<float, float>(a, st) : f32 ? launch_finish<T16, float>(a, st) : launch_finish<T16, T16>(a, st);
}

} // namespace b200p
