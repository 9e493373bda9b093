// ---------------------------------------------------------------------------
// latent_attn.cu -- latent attention (latent.cuh) for a few new tokens on the latent cache,
// in absorbed form on warp MMAs, and the plain kernel for any shape and type.
//
// The absorbed step is four kernels, each a programmatic dependent of the one before:
//  1. absorb: q_abs[h] = W_uk[h]^T q[h] (a weight stream, 16 rows of W_uk^T per warp in registers before the
//     dependency wait); one more CTA normalises the new latents into the cache and rotates their key parts;
//  2. attend: CTA = (sequence, 16 or 32 query rows, split of the keys).  A row is a (token, head); all rows read
//     the same cached vectors, so a tile of 64 keys is loaded once (TMA, 128-byte swizzle) and is keys AND values.
//     For the scores each of the 8 warps takes 8 keys, for the weighted sum a 16-column group of the latents;
//     the weights cross over through shared memory.  Cached tiles are fetched before the dependency wait;
//  3. merge: CTA = (row, 128 latent columns): the splits' partial results and the sink;
//  4. values: CTA = (head, 16 value columns): W_uv (in registers before the dependency wait) and the gate.
// mma.sync: with 16 heads the step does 30 FLOP per byte of cache, far from what needs tcgen05.
// ---------------------------------------------------------------------------
#include "latent.cuh"
#include "attn_common.cuh"
#include "mma_sync.cuh"
#include "vec_io.cuh"
#include "tensor_map.cuh"
#include "dme/dme_tma.cuh"
#include <algorithm>
#include "b200p.h"
#include "wave_primitives/wave64.cuh"

namespace b200p {
namespace {

constexpr int kPlainRows = 8;            // query rows (warps) per CTA
constexpr int kPlainKeys = 32;           // keys per tile: one per lane for the scores

// Causal attention on expanded keys and values in fp32 arithmetic: one warp per query row, one key per lane for
// the scores, one value column per lane (NV of them) for the weighted sum.  Rows and columns come from padded
// buffers, so there is no tail in the dot products.  The gate's sigmoid is applied to the result.
template <typename T, int NV>
__global__ void __launch_bounds__(kPlainRows * 32)
latent_plain_kernel(const LatentAttn a) {
    griddep_launch_dependents();
    extern __shared__ float plain_smem[];
    const LatentDims& d = a.d;
    const int DT = d.dim + d.rot, KS = DT + 1, VD = d.vdim;
    float* sq = plain_smem;                        // [rows][DT]
    float* sk = sq + kPlainRows * DT;              // [keys][DT + 1]
    float* sv = sk + kPlainKeys * KS;              // [keys][VD]
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int h = blockIdx.y, b = blockIdx.z, t0 = blockIdx.x * kPlainRows, t = t0 + warp;
    const int N = a.pos0 + a.Tn;
    const bool live = t < a.Tn;
    const size_t row = size_t(b) * a.Tn + (live ? t : 0);
    const T* q = static_cast<const T*>(a.q) + row * d.q_row() + size_t(h) * DT;
    for (int i = lane; i < DT; i += 32) sq[warp * DT + i] = live ? to_float(q[i]) : 0.f;
    const int last = a.pos0 + t;                                   // newest key this row sees
    const int tile_end = min(a.pos0 + min(t0 + kPlainRows, a.Tn), N);   // keys any row of the CTA sees
    const T* kv = static_cast<const T*>(a.kv) + size_t(b) * N * d.kv_row();
    const T* cache = static_cast<const T*>(a.cache) + size_t(b) * a.max_seq * d.cache_row() + d.rank;
    float acc[NV];
    #pragma unroll
    for (int i = 0; i < NV; ++i) acc[i] = 0.f;
    float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f;
    for (int k0 = 0; k0 < tile_end; k0 += kPlainKeys) {
        __syncthreads();
        for (int i = threadIdx.x; i < kPlainKeys * DT; i += kPlainRows * 32) {
            const int k = i / DT, c = i % DT, n = k0 + k;
            float v = 0.f;
            if (n < N) v = c < d.dim ? to_float(kv[size_t(n) * d.kv_row() + size_t(h) * d.dim + c])
                                     : to_float(cache[size_t(n) * d.cache_row() + c - d.dim]);
            sk[k * KS + c] = v;
        }
        for (int i = threadIdx.x; i < kPlainKeys * VD; i += kPlainRows * 32) {
            const int k = i / VD, c = i % VD, n = k0 + k;
            sv[i] = n < N ? to_float(kv[size_t(n) * d.kv_row() + size_t(d.heads) * d.dim + size_t(h) * VD + c]) : 0.f;
        }
        __syncthreads();
        const float* kr = sk + lane * KS;
        const float* qr = sq + warp * DT;
        float s = 0.f;
        for (int c = 0; c < DT; ++c) s += qr[c] * kr[c];
        s = k0 + lane <= last ? s * a.scale : -INFINITY;
        const float mn = fmaxf(m, wave::dpp::reduce_max(s));
        const float f = m == -INFINITY ? 0.f : expf(m - mn);
        const float p = s == -INFINITY ? 0.f : expf(s - mn);
        l = l * f + wave::dpp::reduce_sum(p);
        m = mn;
        #pragma unroll
        for (int i = 0; i < NV; ++i) acc[i] *= f;
        for (int k = 0; k < kPlainKeys; ++k) {
            const float pk = __shfl_sync(0xffffffffu, p, k);
            #pragma unroll
            for (int i = 0; i < NV; ++i) if (lane + 32 * i < VD) acc[i] += pk * sv[k * VD + lane + 32 * i];
        }
    }
    if (!live) return;
    const float inv = 1.f / l;
    const float* gate = a.proj + row * d.proj_row() + d.gate_col() + size_t(h) * VD;
    T* out = static_cast<T*>(a.out) + row * d.v_row() + size_t(h) * VD;
    #pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = lane + 32 * i;
        if (c < VD) out[c] = from_float<T>(acc[i] * inv / (1.f + expf(-gate[c])));
    }
}

template <typename T, int NV>
int launch_plain(const LatentAttn& a, cudaStream_t st) {
    const size_t smem = (size_t(kPlainRows) * (a.d.dim + a.d.rot) + size_t(kPlainKeys) * (a.d.dim + a.d.rot + 1) + size_t(kPlainKeys) * a.d.vdim) * 4;
    if (smem > 220 * 1024) return B200P_E_DIM;
    auto kern = latent_plain_kernel<T, NV>;
    if (smem > 48 * 1024)
        if (cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem))) return int(e);
    kern<<<dim3(unsigned((a.Tn + kPlainRows - 1) / kPlainRows), unsigned(a.d.heads), unsigned(a.batch)), kPlainRows * 32, smem, st>>>(a);
    return launched();
}

template <typename T>
int launch_plain_t(const LatentAttn& a, cudaStream_t st) {
    if (a.d.vdim <= 32) return launch_plain<T, 1>(a, st);
    if (a.d.vdim <= 64) return launch_plain<T, 2>(a, st);
    if (a.d.vdim <= 128) return launch_plain<T, 4>(a, st);
    if (a.d.vdim <= 256) return launch_plain<T, 8>(a, st);
    if (a.d.vdim <= 512) return launch_plain<T, 16>(a, st);
    return B200P_E_DIM;
}

// ---- the absorbed step ------------------------------------------------------------------------------
using T16 = __nv_bfloat16;
constexpr int kStepThreads = 256, kStepWarps = 8;
constexpr int kAttendKeys = 64;
constexpr float kNegBig = -1e30f;
constexpr int kMaxSplits = 128;          // the merge reads up to four splits per lane

__device__ __forceinline__ int first_pos(const LatentStep& a) { return a.pos_dev ? min(*a.pos_dev, a.max_seq - a.Tn) : a.pos0; }

// Sixteen rows of a weight matrix against X: the A fragments are 32 contiguous bytes of a row per lane (a dot product
// does not care about the order of k): in a 64-column block lane t4 of a row supplies columns 16 t4 .. 16 t4 + 15, and
// reads the same columns of X for the B fragments.  Columns past K are zeros.
struct RowFrag { uint32_t a[8], b[8]; };        // rows g and g + 8
__device__ __forceinline__ void load_rows(RowFrag& f, const T16* w, int ld, int K, int blk, int lane) {
    const int g = lane / 4, c = blk * 64 + (lane % 4) * 16;
    if (c < K) {
        VecIO<32>::load(w + size_t(g) * ld + c, f.a);
        VecIO<32>::load(w + size_t(g + 8) * ld + c, f.b);
    } else {
        #pragma unroll
        for (int i = 0; i < 8; ++i) f.a[i] = f.b[i] = 0u;
    }
}
// x: row g of X (null: zeros), already at column 0
__device__ __forceinline__ void mma_rows(float (&acc)[4], const RowFrag& f, const T16* x, int K, int blk, int lane) {
    const int c = blk * 64 + (lane % 4) * 16;
    uint4 xa = make_uint4(0u, 0u, 0u, 0u), xb = xa;
    if (x && c < K) { xa = *reinterpret_cast<const uint4*>(x + c); xb = *reinterpret_cast<const uint4*>(x + c + 8); }
    const uint32_t xw[8] = {xa.x, xa.y, xa.z, xa.w, xb.x, xb.y, xb.z, xb.w};
    #pragma unroll
    for (int s = 0; s < 4; ++s) {
        const uint32_t af[4] = {f.a[2 * s], f.b[2 * s], f.a[2 * s + 1], f.b[2 * s + 1]};
        mma_16816<T16>(acc, af, xw[2 * s], xw[2 * s + 1]);
    }
}

// 1. grid (rank / 128 rounded up, heads + 1): the last y normalises and caches the new tokens.
template <int MH>
__global__ void __launch_bounds__(kStepThreads) latent_absorb_kernel(const LatentStep a) {
    griddep_launch_dependents();
    const LatentDims& d = a.d;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, M = a.batch * a.Tn;
    if (int(blockIdx.y) == d.heads) {
        if (blockIdx.x != 0) return;
        griddep_wait();
        for (int m = warp; m < M; m += kStepWarps) {
            const float* p = a.proj + size_t(m) * d.proj_row() + d.qrank;
            const T16* w = static_cast<const T16*>(a.kv_norm);
            const int pos = first_pos(a) + m % a.Tn;
            T16* row = static_cast<T16*>(a.cache) + (size_t(m / a.Tn) * a.max_seq + pos) * d.cache_row();
            float ss = 0.f;
            for (int q = lane; q < d.rank / 4; q += 32) {
                const float4 v = *reinterpret_cast<const float4*>(p + 4 * q);
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            }
            const float inv = rsqrtf(wave::dpp::reduce_sum(ss) / a.kv_rank + a.eps);
            for (int q = lane; q < d.rank / 4; q += 32) {
                const float4 v = *reinterpret_cast<const float4*>(p + 4 * q);
                const uint2 wv = *reinterpret_cast<const uint2*>(w + 4 * q);
                const T16* g = reinterpret_cast<const T16*>(&wv);
                *reinterpret_cast<uint2*>(row + 4 * q) = make_uint2(pack2<T16>(v.x * inv * to_float(g[0]), v.y * inv * to_float(g[1])),
                                                                    pack2<T16>(v.z * inv * to_float(g[2]), v.w * inv * to_float(g[3])));
            }
            const float* k = p + d.rank;
            for (int i = lane; i < d.rot / 2; i += 32) {
                const int u = 16 * (i / 8) + i % 8;
                const size_t t = size_t(pos) * (d.rot / 2) + i;
                const float c = a.cos_t[t], sn = a.sin_t[t], x0 = k[u], x1 = k[u + 8];
                row[d.rank + u] = from_float<T16>(x0 * c - x1 * sn);
                row[d.rank + u + 8] = from_float<T16>(x1 * c + x0 * sn);
            }
        }
        return;
    }
    const int h = blockIdx.y, r0 = (blockIdx.x * kStepWarps + warp) * 16;       // 16 rows of W_uk[h]^T
    if (r0 >= d.rank) return;
    const T16* w = static_cast<const T16*>(a.ukT) + (size_t(h) * d.rank + r0) * d.dim;
    const int nblk = (d.dim + 63) / 64;
    RowFrag f0, f1;
    load_rows(f0, w, d.dim, d.dim, 0, lane);
    if (nblk > 1) load_rows(f1, w, d.dim, d.dim, 1, lane);
    griddep_wait();
    const int g = lane / 4, t4 = lane % 4;
    #pragma unroll
    for (int mh = 0; mh < MH; ++mh) {
        const int mx = 8 * mh + g;
        const T16* x = mx < M ? static_cast<const T16*>(a.q_plain) + size_t(mx) * d.heads * d.dim + size_t(h) * d.dim : nullptr;
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        mma_rows(acc, f0, x, d.dim, 0, lane);
        if (nblk > 1) mma_rows(acc, f1, x, d.dim, 1, lane);
        for (int b = 2; b < nblk; ++b) {
            RowFrag f;
            load_rows(f, w, d.dim, d.dim, b, lane);
            mma_rows(acc, f, x, d.dim, b, lane);
        }
        #pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int m = 8 * mh + 2 * t4 + (c & 1), r = r0 + g + 8 * (c >> 1);
            if (m < M) static_cast<T16*>(a.q_abs)[(size_t(m) * d.heads + h) * d.cache_row() + r] = from_float<T16>(acc[c]);
        }
    }
}

// Keys of this step and of a split (whole tiles); every kernel of the step derives the same.
__device__ __forceinline__ void step_extent(const LatentStep& a, int splits, int& N, int& per) {
    N = first_pos(a) + a.Tn;
    per = ((N + splits - 1) / splits + kAttendKeys - 1) / kAttendKeys * kAttendKeys;
}

// Shared memory of the attend kernel: tiles of `boxes` boxes [64 keys][128 B] in a ring of `stages`, the query rows in
// boxes [16 MT rows][128 B], the weights [16 MT rows][64 keys].
template <int MT> struct AttendSmem {
    static constexpr int ROWS = 16 * MT;
    int boxes, stages;
    __host__ __device__ int tile() const { return boxes * kAttendKeys * 128; }
    __host__ __device__ int q() const { return stages * tile(); }
    __host__ __device__ int p() const { return q() + boxes * ROWS * 128; }
    __host__ __device__ int total() const { return p() + ROWS * 128; }
};

// NG: 16-column groups of the latents per warp.
template <int MT, int NG>
__global__ void __launch_bounds__(kStepThreads + 32, 1)
latent_attend_kernel(const LatentStep a, const __grid_constant__ CUtensorMap map, int splits, int stages, int* sticky) {
    griddep_launch_dependents();
    constexpr int ROWS = 16 * MT;
    extern __shared__ __align__(1024) unsigned char attend_smem[];
    __shared__ float s_max[kStepWarps][ROWS];
    __shared__ float s_sum[kStepWarps][ROWS];
    __shared__ uint64_t bars[16];
    __shared__ int s_failed;
    const LatentDims& d = a.d;
    const int C = d.cache_row(), boxes = (C + 63) / 64;
    const AttendSmem<MT> sm{boxes, stages};
    uint64_t* full = bars;
    uint64_t* empty = bars + 8;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int split = blockIdx.x, b = blockIdx.z;
    const int R = a.Tn * d.heads, row0 = blockIdx.y * ROWS;        // rows of the sequence, this CTA's first
    if (threadIdx.x == 0) {
        s_failed = 0;
        for (int s = 0; s < stages; ++s) { dme::mbar_init(&full[s], 1); dme::mbar_init(&empty[s], kStepWarps); }
        dme::mbar_init_fence();
    }
    __syncthreads();
    int N, per;
    step_extent(a, splits, N, per);
    const int old = N - a.Tn;                                       // rows of the cache from before this step
    const int k0 = min(split * per, N), k1 = min(k0 + per, N);
    const int ntiles = (k1 - k0 + kAttendKeys - 1) / kAttendKeys;
    if (warp == kStepWarps) {
        if (lane == 0) {
            dme::prefetch_tensor_map(&map);
            int stage = 0; uint32_t phase = 0;
            bool waited = false;
            for (int t = 0; t < ntiles; ++t) {
                const int key = k0 + t * kAttendKeys;
                if (!waited && key + kAttendKeys > old) { griddep_wait(); waited = true; }      // the tile holds new keys
                if (t >= stages && !dme::wait(&empty[stage], phase ^ 1u, a.abort_word)) { atomicExch(&s_failed, 1); break; }
                dme::mbar_arrive_expect_tx(&full[stage], uint32_t(sm.tile()));
                unsigned char* dst = attend_smem + stage * sm.tile();
                for (int x = 0; x < boxes; ++x)
                    dme::copy_tile_2d(dst + x * kAttendKeys * 128, &map, x * 64, b * a.max_seq + key, &full[stage]);
                if (++stage == stages) { stage = 0; phase ^= 1u; }
            }
        }
    } else {
        griddep_wait();
        const int g = lane / 4, t4 = lane % 4, mi = lane / 8, r8 = lane % 8;
        auto sync = [] { asm volatile("bar.sync 1, %0;" :: "n"(kStepThreads) : "memory"); };
        // query rows into swizzled boxes, zeros past the rows and columns that exist
        unsigned char* qs = attend_smem + sm.q();
        unsigned char* ps = attend_smem + sm.p();
        for (int i = threadIdx.x; i < ROWS * boxes * 8; i += kStepThreads) {
            const int r = i / (boxes * 8), ch = i % (boxes * 8);
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (row0 + r < R && ch * 8 < C)
                v = *reinterpret_cast<const uint4*>(static_cast<const T16*>(a.q_abs) + (size_t(b) * R + row0 + r) * C + ch * 8);
            *reinterpret_cast<uint4*>(qs + (ch >> 3) * (ROWS * 128) + swz128(r, ch & 7)) = v;
        }
        sync();
        const uint32_t qa = dme::smem_addr(qs), pa = dme::smem_addr(ps);
        const float scale_log2 = a.scale * 1.4426950408889634f;
        float o[MT][NG][2][4];
        float m[MT][2], l[MT][2];
        int limit[MT][2];                                           // newest key the row sees
        #pragma unroll
        for (int t = 0; t < MT; ++t) {
            #pragma unroll
            for (int i = 0; i < NG; ++i)
                #pragma unroll
                for (int j = 0; j < 4; ++j) o[t][i][0][j] = o[t][i][1][j] = 0.f;
            #pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                m[t][hf] = kNegBig; l[t][hf] = 0.f;
                limit[t][hf] = old + min(row0 + 16 * t + 8 * hf + g, R - 1) / d.heads;
            }
        }
        const int ngroups = d.rank / 16;
        int stage = 0; uint32_t phase = 0;
        bool ok = true;
        for (int t = 0; t < ntiles; ++t) {
            // (a wait that gave up: the warps go on through the barriers together, without the tile)
            if (ok && !dme::wait(&full[stage], phase, a.abort_word)) { ok = false; atomicExch(&s_failed, 1); }
            ok = __all_sync(0xffffffffu, ok);
            const uint32_t kt = dme::smem_addr(attend_smem + stage * sm.tile());
            // ---- scores of this warp's 8 keys ------------------------------------------------------------
            float s[MT][4][4];
            #pragma unroll
            for (int x = 0; x < MT; ++x)
                #pragma unroll
                for (int c = 0; c < 4; ++c) s[x][c][0] = s[x][c][1] = s[x][c][2] = s[x][c][3] = 0.f;
            if (ok) {
                #pragma unroll(MT == 1 ? 3 : 1)
                for (int bx = 0; bx < boxes; ++bx) {                // 64 columns: four k-steps, one accumulator each
                    const uint32_t kb = kt + bx * (kAttendKeys * 128), qb = qa + bx * (ROWS * 128);
                    uint32_t bk[2][4];
                    ldmatrix_x4(bk[0], kb + swz128(8 * warp + r8, mi));
                    ldmatrix_x4(bk[1], kb + swz128(8 * warp + r8, 4 + mi));
                    #pragma unroll
                    for (int ks = 0; ks < 4; ++ks) {
                        #pragma unroll
                        for (int x = 0; x < MT; ++x) {
                            uint32_t aq[4];
                            ldmatrix_x4(aq, qb + swz128(16 * x + (mi & 1) * 8 + r8, 2 * ks + (mi >> 1)));
                            mma_16816<T16>(s[x][ks], aq, bk[ks >> 1][2 * (ks & 1)], bk[ks >> 1][2 * (ks & 1) + 1]);
                        }
                    }
                }
            }
            const int key = k0 + t * kAttendKeys + 8 * warp + 2 * t4;
            float sc[MT][4];
            #pragma unroll
            for (int x = 0; x < MT; ++x) {
                #pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float v = (s[x][0][j] + s[x][1][j]) + (s[x][2][j] + s[x][3][j]);
                    sc[x][j] = key + (j & 1) <= limit[x][j >> 1] && key + (j & 1) < k1 ? v * scale_log2 : kNegBig;
                }
                #pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const float mx = wave::lane_group_reduce<4>(fmaxf(sc[x][2 * hf], sc[x][2 * hf + 1]), wave::MaxOp{});
                    if (t4 == 0) s_max[warp][16 * x + 8 * hf + g] = mx;
                }
            }
            sync();
            // ---- running maxima over all warps' keys, weights into shared memory ------------------------------
            bool moved = false;
            float alpha[MT][2];
            #pragma unroll
            for (int x = 0; x < MT; ++x) {
                #pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const int r = 16 * x + 8 * hf + g;
                    const float mx = wave::lane_group_reduce<4>(fmaxf(s_max[2 * t4][r], s_max[2 * t4 + 1][r]), wave::MaxOp{});
                    const float mn = fmaxf(m[x][hf], mx);
                    alpha[x][hf] = fast_exp2(m[x][hf] - mn);
                    moved |= mn != m[x][hf];
                    m[x][hf] = mn;
                    const float p0 = sc[x][2 * hf] > kNegBig ? fast_exp2(sc[x][2 * hf] - mn) : 0.f;
                    const float p1 = sc[x][2 * hf + 1] > kNegBig ? fast_exp2(sc[x][2 * hf + 1] - mn) : 0.f;
                    l[x][hf] = l[x][hf] * alpha[x][hf] + p0 + p1;
                    *reinterpret_cast<uint32_t*>(ps + swz128(r, warp) + 4 * t4) = pack2<T16>(p0, p1);
                }
            }
            if (__any_sync(0xffffffffu, moved)) {
                #pragma unroll
                for (int x = 0; x < MT; ++x)
                    #pragma unroll
                    for (int i = 0; i < NG; ++i)
                        #pragma unroll
                        for (int n = 0; n < 2; ++n)
                            #pragma unroll
                            for (int j = 0; j < 4; ++j) o[x][i][n][j] *= alpha[x][j >> 1];
            }
            sync();
            // ---- weighted sum of the latents: this warp's column groups ------------------------------------------
            if (ok) {
                #pragma unroll
                for (int ks = 0; ks < kAttendKeys / 16; ++ks) {
                    uint32_t ap[MT][4];
                    #pragma unroll
                    for (int x = 0; x < MT; ++x) ldmatrix_x4(ap[x], pa + swz128(16 * x + (mi & 1) * 8 + r8, 2 * ks + (mi >> 1)));
                    #pragma unroll
                    for (int i = 0; i < NG; ++i) {
                        const int grp = warp + kStepWarps * i;
                        if (grp < ngroups) {                        // warp-uniform
                            uint32_t bv[4];
                            const int chunk = 2 * grp + (mi >> 1);
                            ldmatrix_x4_trans(bv, kt + (chunk >> 3) * (kAttendKeys * 128) + swz128(16 * ks + (mi & 1) * 8 + r8, chunk & 7));
                            #pragma unroll
                            for (int x = 0; x < MT; ++x) {
                                mma_16816<T16>(o[x][i][0], ap[x], bv[0], bv[1]);
                                mma_16816<T16>(o[x][i][1], ap[x], bv[2], bv[3]);
                            }
                        }
                    }
                }
            }
            __syncwarp();
            if (lane == 0) dme::mbar_arrive(&empty[stage]);
            if (++stage == stages) { stage = 0; phase ^= 1u; }
        }
        // ---- partial results of the split: columns by warp, sums over the warps' keys --------------------------
        #pragma unroll
        for (int x = 0; x < MT; ++x) {
            #pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const float ls = wave::lane_group_reduce<4>(l[x][hf], wave::SumOp{});
                if (t4 == 0) s_sum[warp][16 * x + 8 * hf + g] = ls;
                const int r = row0 + 16 * x + 8 * hf + g;
                if (r >= R) continue;
                float* po = a.part_o + ((size_t(b) * R + r) * splits + split) * d.rank;
                #pragma unroll
                for (int i = 0; i < NG; ++i) {
                    const int grp = warp + kStepWarps * i;
                    if (grp < ngroups) {
                        *reinterpret_cast<float2*>(po + grp * 16 + 2 * t4) = make_float2(o[x][i][0][2 * hf], o[x][i][0][2 * hf + 1]);
                        *reinterpret_cast<float2*>(po + grp * 16 + 8 + 2 * t4) = make_float2(o[x][i][1][2 * hf], o[x][i][1][2 * hf + 1]);
                    }
                }
            }
        }
        sync();
        if (warp == 0 && t4 == 0) {
            #pragma unroll
            for (int x = 0; x < MT; ++x) {
                #pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const int rl = 16 * x + 8 * hf + g;
                    float ls = 0.f;
                    #pragma unroll
                    for (int w = 0; w < kStepWarps; ++w) ls += s_sum[w][rl];
                    if (row0 + rl < R)
                        *reinterpret_cast<float2*>(a.part_ml + 2 * ((size_t(b) * R + row0 + rl) * splits + split)) = make_float2(m[x][hf], ls);
                }
            }
        }
    }
    __syncthreads();
    if (threadIdx.x == 0 && s_failed) { atomicExch(a.abort_word, 1); atomicExch(sticky, 1); }
}

// 3. grid (rows, rank / 128 rounded up): merges the splits of a row.  A split's share is e^(m_s - m) / l, with the sink as
// one more term of l.  One warp per split in turn, four columns per lane.
__global__ void __launch_bounds__(kStepThreads) latent_merge_kernel(const LatentStep a, int splits) {
    griddep_launch_dependents();
    __shared__ float s_w[kMaxSplits];
    __shared__ float4 part[kStepWarps][32];
    const LatentDims& d = a.d;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, h = blockIdx.x % d.heads;
    const size_t row = blockIdx.x;
    const int c = (blockIdx.y * 32 + lane) * 4;
    griddep_wait();
    int N, per;
    step_extent(a, splits, N, per);
    const int used = (N + per - 1) / per;                           // splits with keys
    if (warp == 0) {
        constexpr int PER = kMaxSplits / 32;
        const float sink = a.sink ? a.sink[h] * 1.4426950408889634f : kNegBig;
        float2 ml[PER];
        float top = sink;
        #pragma unroll
        for (int i = 0; i < PER; ++i) {
            ml[i] = make_float2(kNegBig, 0.f);
            if (lane + 32 * i < used) ml[i] = *reinterpret_cast<const float2*>(a.part_ml + 2 * (row * splits + lane + 32 * i));
            top = fmaxf(top, ml[i].x);
        }
        top = wave::dpp::reduce_max(top);
        float l = 0.f;
        #pragma unroll
        for (int i = 0; i < PER; ++i) { ml[i].x = fast_exp2(ml[i].x - top); l += ml[i].x * ml[i].y; }
        l = wave::dpp::reduce_sum(l);
        if (a.sink) l += fast_exp2(sink - top);
        #pragma unroll
        for (int i = 0; i < PER; ++i) if (lane + 32 * i < used) s_w[lane + 32 * i] = ml[i].x / l;
    }
    float4 v[8];                                                    // the first splits' columns, on their way meanwhile
    const float* po = a.part_o + row * splits * d.rank + c;
    const bool live = c < d.rank;
    #pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int sp = warp + kStepWarps * i;
        v[i] = live && sp < used ? *reinterpret_cast<const float4*>(po + size_t(sp) * d.rank) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    __syncthreads();
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    auto take = [&](const float4& x, int sp) {
        const float f = s_w[sp];
        acc.x += f * x.x; acc.y += f * x.y; acc.z += f * x.z; acc.w += f * x.w;
    };
    #pragma unroll
    for (int i = 0; i < 8; ++i) if (warp + kStepWarps * i < used) take(v[i], warp + kStepWarps * i);
    for (int sp = warp + kStepWarps * 8; sp < used; sp += kStepWarps)
        if (live) take(*reinterpret_cast<const float4*>(po + size_t(sp) * d.rank), sp);
    part[warp][lane] = acc;
    __syncthreads();
    if (warp == 0 && live) {
        #pragma unroll
        for (int w = 1; w < kStepWarps; ++w) { const float4 x = part[w][lane]; acc.x += x.x; acc.y += x.y; acc.z += x.z; acc.w += x.w; }
        *reinterpret_cast<uint2*>(static_cast<T16*>(a.merged) + row * d.rank + c) = make_uint2(pack2<T16>(acc.x, acc.y), pack2<T16>(acc.z, acc.w));
    }
}

// 4. grid (vdim / 16, heads): W_uv and the gate.
template <int MH>
__global__ void __launch_bounds__(kStepThreads) latent_values_kernel(const LatentStep a) {
    griddep_launch_dependents();
    __shared__ float red[kStepWarps][32][4 * MH];
    const LatentDims& d = a.d;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, M = a.batch * a.Tn;
    const int h = blockIdx.y, v0 = blockIdx.x * 16;
    const T16* w = static_cast<const T16*>(a.uv) + (size_t(h) * d.vdim + v0) * d.rank;
    const int nblk = (d.rank + 63) / 64;                            // 64-column blocks, dealt to the warps
    RowFrag f0;
    if (warp < nblk) load_rows(f0, w, d.rank, d.rank, warp, lane);
    griddep_wait();
    float gate[MH];                                                 // for the epilogue, on their way during the product
    if (threadIdx.x < 128) {
        #pragma unroll
        for (int mh = 0; mh < MH; ++mh) {
            const int m = 8 * mh + 2 * (lane % 4) + (warp & 1), n = v0 + lane / 4 + 8 * (warp >> 1);
            gate[mh] = m < M ? a.proj[size_t(m) * d.proj_row() + d.gate_col() + size_t(h) * d.vdim + n] : 0.f;
        }
    }
    const int g = lane / 4;
    #pragma unroll
    for (int mh = 0; mh < MH; ++mh) {
        const int mx = 8 * mh + g;
        const T16* x = mx < M ? static_cast<const T16*>(a.merged) + (size_t(mx) * d.heads + h) * d.rank : nullptr;
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        if (warp < nblk) mma_rows(acc, f0, x, d.rank, warp, lane);
        for (int blk = warp + kStepWarps; blk < nblk; blk += kStepWarps) {
            RowFrag f;
            load_rows(f, w, d.rank, d.rank, blk, lane);
            mma_rows(acc, f, x, d.rank, blk, lane);
        }
        *reinterpret_cast<float4*>(&red[warp][lane][4 * mh]) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    }
    __syncthreads();
    if (threadIdx.x < 128) {
        #pragma unroll
        for (int mh = 0; mh < MH; ++mh) {
            float v = 0.f;
            #pragma unroll
            for (int k = 0; k < kStepWarps; ++k) v += red[k][lane][4 * mh + warp];
            const int m = 8 * mh + 2 * (lane % 4) + (warp & 1), n = v0 + lane / 4 + 8 * (warp >> 1);
            if (m < M) static_cast<T16*>(a.out)[size_t(m) * d.v_row() + size_t(h) * d.vdim + n] = from_float<T16>(v / (1.f + expf(-gate[mh])));
        }
    }
}

// How the keys and rows of a step are cut; depends on nothing that changes from step to step.
struct StepPlan { int mt, groups, splits, stages; size_t smem; };
template <int MT> size_t attend_bytes(int boxes, int stages) { return size_t(AttendSmem<MT>{boxes, stages}.total()); }
StepPlan step_plan(const LatentDims& d, int batch, int Tn) {
    StepPlan p{};
    const int R = Tn * d.heads, boxes = (d.cache_row() + 63) / 64, sms = std::max(sm_count(), 1);
    p.mt = R <= 16 ? 1 : 2;
    p.groups = (R + 16 * p.mt - 1) / (16 * p.mt);
    const int want = tuning(KNOB_DECODE_SPLITS, 0);                 // 0: as below
    p.splits = std::max(1, std::min(want > 0 ? std::min(want, kMaxSplits) : 64, sms / (p.groups * batch)));
    for (p.stages = 4; p.stages >= 2; --p.stages) {
        p.smem = p.mt == 1 ? attend_bytes<1>(boxes, p.stages) : attend_bytes<2>(boxes, p.stages);
        if (p.smem <= 220 * 1024) break;
    }
    return p;                                                        // stages < 2: does not fit
}

template <int MT, int NG>
int launch_attend(const LatentStep& a, const StepPlan& p, cudaStream_t st) {
    CUtensorMap map;
    const LatentDims& d = a.d;
    const uint64_t dims[2] = {uint64_t(d.cache_row()), uint64_t(a.batch) * a.max_seq}, strides[1] = {uint64_t(d.cache_row()) * 2};
    const uint32_t box[2] = {64, kAttendKeys};
    if (cudaError_t e = make_tensor_map(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.cache, dims, strides, box, Swizzle::B128)) return int(e);
    int* sticky = device_status_ptr();
    if (!sticky) return B200P_E_NO_DEVICE;
    auto kern = latent_attend_kernel<MT, NG>;
    if (cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(p.smem))) return int(e);
    return launch_dependent(kern, dim3(unsigned(p.splits), unsigned(p.groups), unsigned(a.batch)), kStepThreads + 32, p.smem, st, a, map, p.splits, p.stages, sticky);
}

} // namespace

int latent_attn_plain(const LatentAttn& a, cudaStream_t st) {
    if (a.d.heads > 65535 || a.batch > 65535) return B200P_E_RANGE;
    return a.dtype == B200P_F32 ? launch_plain_t<float>(a, st) : launch_plain_t<__nv_bfloat16>(a, st);
}

bool latent_step_ok(const LatentDims& d, int M) {
    return M <= 16 && d.rank <= 512 && d.heads < 65535 && step_plan(d, 1, M).stages >= 2;
}
// splits * rows of a step is at most this many: the splits only multiply until the row groups fill the SMs
size_t latent_step_partials(const LatentDims& d) { return std::max(size_t(16) * d.heads, size_t(std::max(sm_count(), 1)) * 32); }

int latent_step_absorb(const LatentStep& a, cudaStream_t st) {
    const dim3 grid(unsigned((a.d.rank + 16 * kStepWarps - 1) / (16 * kStepWarps)), unsigned(a.d.heads + 1));
    return launch_dependent(a.batch * a.Tn <= 8 ? latent_absorb_kernel<1> : latent_absorb_kernel<2>, grid, kStepThreads, 0, st, a);
}

int latent_step_attend(const LatentStep& a, cudaStream_t st) {
    const StepPlan p = step_plan(a.d, a.batch, a.Tn);
    if (p.stages < 2 || a.d.rank > 512) return B200P_E_RANGE;
    const int ng = (a.d.rank / 16 + kStepWarps - 1) / kStepWarps;
    if (p.mt == 1) return ng <= 1 ? launch_attend<1, 1>(a, p, st) : ng <= 2 ? launch_attend<1, 2>(a, p, st) : launch_attend<1, 4>(a, p, st);
    return ng <= 1 ? launch_attend<2, 1>(a, p, st) : ng <= 2 ? launch_attend<2, 2>(a, p, st) : launch_attend<2, 4>(a, p, st);
}

int latent_step_values(const LatentStep& a, cudaStream_t st) {
    const int M = a.batch * a.Tn;
    const StepPlan p = step_plan(a.d, a.batch, a.Tn);
    if (int e = launch_dependent(latent_merge_kernel, dim3(unsigned(M * a.d.heads), unsigned((a.d.rank + 127) / 128)), kStepThreads, 0, st, a, p.splits)) return e;
    return launch_dependent(M <= 8 ? latent_values_kernel<1> : latent_values_kernel<2>, dim3(unsigned(a.d.vdim / 16), unsigned(a.d.heads)), kStepThreads, 0, st, a);
}

} // namespace b200p
