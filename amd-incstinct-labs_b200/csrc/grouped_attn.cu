// ---------------------------------------------------------------------------
// grouped_attn.cu -- grouped attention (grouped_attn.cuh): a projection's rows into queries and
// the cache, the plain kernel for any shape and type, and the decode step's kernel.
//
// grouped_step takes one new token per sequence from the fp32 projection to the gated output in
// one launch.  A cluster is a (sequence, key/value head, 16 query heads), its CTAs split the keys
// that the mask leaves:
//   * the cached keys and values stream through a TMA ring (128 keys a stage, 64-column boxes,
//     128-byte swizzle) and are asked for BEFORE the dependency wait: all of them were written by
//     earlier steps.  The new key never goes through the cache on its way to the score: it is
//     rotated and normalised in registers and joins the merge as a ninth partial result, as the
//     softmax's extra term does;
//   * the query heads of the group are the 16 rows of mma.sync m16n8k16, a warp takes 16 keys of
//     a stage (decode_mma_kernel's scheme);
//   * the CTAs' partial results meet in distributed shared memory, each CTA finishes its share of
//     the output columns: no partials in global memory, no ticket, no second launch.
// ---------------------------------------------------------------------------
#include "grouped_attn.cuh"
#include "mma_sync.cuh"
#include "tensor_map.cuh"
#include "vec_quads.cuh"
#include "dme/dme_tma.cuh"
#include "wave_primitives/wave64.cuh"
#include "b200p.h"
#include <algorithm>
#include <cooperative_groups.h>

namespace b200p {
namespace {
namespace cg = cooperative_groups;

constexpr float kLog2e = 1.4426950408889634f;
constexpr float kNegBig = -1e30f;

// ---- the projection's rows ------------------------------------------------------------------------------
// Columns col .. col + 3 of a head at position pos: two adjacent pairs turned by their angles.
__device__ __forceinline__ float4 rotate_quad(const float4& v, const GroupedAttn& a, int pos, int col) {
    const size_t t = size_t(pos) * (a.d.dim / 2) + col / 2;
    const float2 c = *reinterpret_cast<const float2*>(a.cos_t + t), s = *reinterpret_cast<const float2*>(a.sin_t + t);
    return make_float4(v.x * c.x - v.y * s.x, v.y * c.x + v.x * s.x, v.z * c.y - v.w * s.y, v.w * c.y + v.z * s.y);
}
__device__ __forceinline__ float dot4(const float4& x, const float4& y) { return (x.x * y.x + x.y * y.y) + (x.z * y.z + x.w * y.w); }
__device__ __forceinline__ float4 scaled(const float4& v, float f) { return make_float4(v.x * f, v.y * f, v.z * f, v.w * f); }

// A group of W lanes per (token, head), eight columns a lane: key heads to the cache (and the values, own or the keys as
// projected); query heads, where something happens to them, in place.
template <typename T, int W, int CH>
__global__ void __launch_bounds__(256) grouped_inputs_kernel(const GroupedAttn a, unsigned units, int slots) {
    const GroupedDims& d = a.d;
    const unsigned u = (blockIdx.x * 256u + threadIdx.x) / W;
    const int c0 = threadIdx.x % W * 8;
    const bool live = u < units;
    const unsigned row = (live ? u : 0) / unsigned(slots);
    const int slot = int((live ? u : 0) - row * slots) + (d.heads + d.kv_heads - slots);          // without queries: the keys only
    const unsigned b = row / unsigned(a.Tn);
    const int pos = a.pos0 + int(row - b * a.Tn), kvh = slot - d.heads;
    T* p = static_cast<T*>(const_cast<void*>(a.proj)) + size_t(row) * d.proj_row();
    T* src = p + slot * d.dim;
    const size_t cache_row = (size_t(b) * d.kv_heads + kvh) * a.max_seq + pos;
    T* dst = kvh >= 0 ? static_cast<T*>(a.kcache) + cache_row * d.dim : src;
    T* vrow = static_cast<T*>(a.vcache) + cache_row * d.vdim;
    float v[CH][8];
    float ss = 0.f;
    #pragma unroll
    for (int i = 0; i < CH; ++i) {
        const int c = c0 + 8 * W * i;
        if (live && c < d.dim) {
            load8<T>(src + c, v[i]);
            #pragma unroll
            for (int k = 0; k < 8; ++k) ss += v[i][k] * v[i][k];
            if (kvh >= 0 && !d.own_values) store8<T>(vrow + c, v[i]);
        }
    }
    if (live && kvh >= 0 && d.own_values)
        for (int c = c0; c < d.vdim; c += 8 * W) {
            float x[8];
            load8<T>(p + d.v_col() + kvh * d.vdim + c, x);
            store8<T>(vrow + c, x);
        }
    // (turning a pair does not change its length: the mean square is the same before and after)
    const float f = a.norm ? rsqrtf(wave::lane_group_reduce<W>(ss, wave::SumOp{}) / d.n_dim + a.eps) : 1.f;
    #pragma unroll
    for (int i = 0; i < CH; ++i) {
        const int c = c0 + 8 * W * i;
        if (!live || c >= d.dim) continue;
        if (a.cos_t) {
            const size_t t = size_t(pos) * (d.dim / 2) + c / 2;
            const float4 cs = load4<float>(a.cos_t + t), sn = load4<float>(a.sin_t + t);
            const float cf[4] = {cs.x, cs.y, cs.z, cs.w}, sf[4] = {sn.x, sn.y, sn.z, sn.w};
            #pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float x = v[i][2 * k], y = v[i][2 * k + 1];
                v[i][2 * k] = x * cf[k] - y * sf[k];
                v[i][2 * k + 1] = y * cf[k] + x * sf[k];
            }
        }
        #pragma unroll
        for (int k = 0; k < 8; ++k) v[i][k] *= f;
        store8<T>(dst + c, v[i]);
    }
}

template <typename T>
int launch_inputs(const GroupedAttn& a, cudaStream_t st) {
    const int slots = (a.cos_t || a.norm ? a.d.heads : 0) + a.d.kv_heads, lanes = a.d.dim / 8;
    const long long units = (long long)a.batch * a.Tn * slots;
    if (units * 32 > 0xffffffffLL) return B200P_E_RANGE;
    auto run = [&](auto kern, int W) {
        kern<<<unsigned((units * W + 255) / 256), 256, 0, st>>>(a, unsigned(units), slots);
        return launched();
    };
    if (lanes <= 2) return run(grouped_inputs_kernel<T, 2, 1>, 2);
    if (lanes <= 4) return run(grouped_inputs_kernel<T, 4, 1>, 4);
    if (lanes <= 8) return run(grouped_inputs_kernel<T, 8, 1>, 8);
    if (lanes <= 16) return run(grouped_inputs_kernel<T, 16, 1>, 16);
    return run(grouped_inputs_kernel<T, 32, 2>, 32);
}

// ---- any shape, fp32 arithmetic ---------------------------------------------------------------------------
constexpr int kPlainRows = 8;            // query rows (warps) per CTA
constexpr int kPlainKeys = 32;           // keys per tile: one per lane for the scores

template <typename T, int NV>
__global__ void __launch_bounds__(kPlainRows * 32) grouped_plain_kernel(const GroupedAttn a) {
    extern __shared__ float plain_smem[];
    const GroupedDims& d = a.d;
    const int DT = d.dim, KS = DT + 1, VD = d.vdim;
    float* sq = plain_smem;                        // [rows][DT]
    float* sk = sq + kPlainRows * DT;              // [keys][DT + 1]
    float* sv = sk + kPlainKeys * KS;              // [keys][VD]
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int h = blockIdx.y, b = blockIdx.z, t0 = blockIdx.x * kPlainRows, t = t0 + warp;
    const bool live = t < a.Tn;
    const size_t row = size_t(b) * a.Tn + (live ? t : 0);
    const T* q = static_cast<const T*>(a.proj) + row * d.proj_row() + size_t(h) * DT;
    for (int i = lane; i < DT; i += 32) sq[warp * DT + i] = live ? to_float(q[i]) : 0.f;
    const int last = a.pos0 + t, first = a.mask.first(last);                 // keys this row sees
    const int end = a.pos0 + min(t0 + kPlainRows, a.Tn);                     // keys any row of the CTA sees: [begin, end)
    const int begin = a.mask.first(a.pos0 + t0);
    const size_t head = size_t(b) * d.kv_heads + h / d.group();
    const T* kc = static_cast<const T*>(a.kcache) + head * a.max_seq * DT;
    const T* vc = static_cast<const T*>(a.vcache) + head * a.max_seq * VD;
    float acc[NV];
    #pragma unroll
    for (int i = 0; i < NV; ++i) acc[i] = 0.f;
    float m = a.plus_one ? 0.f : -INFINITY, l = a.plus_one ? 1.f : 0.f;
    for (int k0 = begin; k0 < end; k0 += kPlainKeys) {
        __syncthreads();
        for (int i = threadIdx.x; i < kPlainKeys * DT; i += kPlainRows * 32) {
            const int k = i / DT, c = i % DT;
            sk[k * KS + c] = k0 + k < end ? to_float(kc[size_t(k0 + k) * DT + c]) : 0.f;
        }
        for (int i = threadIdx.x; i < kPlainKeys * VD; i += kPlainRows * 32) {
            const int k = i / VD, c = i % VD;
            sv[i] = k0 + k < end ? to_float(vc[size_t(k0 + k) * VD + c]) : 0.f;
        }
        __syncthreads();
        const float* kr = sk + lane * KS;
        const float* qr = sq + warp * DT;
        float s = 0.f;
        for (int c = 0; c < DT; ++c) s += qr[c] * kr[c];
        s = k0 + lane >= first && k0 + lane <= last ? s * a.scale : -INFINITY;
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
    const T* gate = d.gated ? static_cast<const T*>(a.proj) + row * d.proj_row() + d.g_col() + size_t(h) * VD : nullptr;
    T* out = static_cast<T*>(a.out) + row * d.v_row() + size_t(h) * VD;
    #pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = lane + 32 * i;
        if (c < VD) out[c] = from_float<T>(gate ? acc[i] * inv / (1.f + expf(-to_float(gate[c]))) : acc[i] * inv);
    }
}

template <typename T, int NV>
int launch_plain(const GroupedAttn& a, cudaStream_t st) {
    const size_t smem = (size_t(kPlainRows) * a.d.dim + size_t(kPlainKeys) * (a.d.dim + 1) + size_t(kPlainKeys) * a.d.vdim) * 4;
    auto kern = grouped_plain_kernel<T, NV>;
    if (smem > 48 * 1024)
        if (cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem))) return int(e);
    kern<<<dim3(unsigned((a.Tn + kPlainRows - 1) / kPlainRows), unsigned(a.d.heads), unsigned(a.batch)), kPlainRows * 32, smem, st>>>(a);
    return launched();
}

template <typename T>
int launch_plain_t(const GroupedAttn& a, cudaStream_t st) {
    if (a.d.vdim <= 64) return launch_plain<T, 2>(a, st);
    if (a.d.vdim <= 128) return launch_plain<T, 4>(a, st);
    return launch_plain<T, 16>(a, st);
}

// ---- one new token per sequence ---------------------------------------------------------------------------
using T16 = __nv_bfloat16;
constexpr int kStepThreads = 256, kStepWarps = 8, kStepKeys = 128, kStepRows = 16;

template <int QKS, int VS> struct StepSmem {
    static constexpr int DV = 64 * VS, BOX = kStepKeys * 128;
    static constexpr int STAGE = (QKS + VS) * BOX, STAGES = QKS + VS > 3 ? 3 : 4;
    static constexpr int OFF_Q = STAGES * STAGE;                            // query rows, boxes [16][128 B]
    static constexpr int OFF_PART = OFF_Q + QKS * kStepRows * 128;          // this CTA's partial result [16][DV]
    static constexpr int BYTES = OFF_PART + kStepRows * DV * 4;
    static constexpr int DP = DV + 8;                                       // merge rows: 8-byte stores on different banks
    static_assert(kStepWarps * kStepRows * (DP + 2) * 4 <= STAGES * STAGE, "the warps' results fit the ring");
};

template <int QKS, int VS>
__global__ void __launch_bounds__(kStepThreads + 32, 1)
grouped_step_kernel(const GroupedAttn a, const __grid_constant__ CUtensorMap mapK, const __grid_constant__ CUtensorMap mapV, int row_tiles, int* sticky) {
    griddep_launch_dependents();
    using Sh = StepSmem<QKS, VS>;
    constexpr int STAGES = Sh::STAGES, DV = Sh::DV, KS = 4 * QKS, DP = Sh::DP;
    extern __shared__ __align__(1024) unsigned char step_smem[];
    __shared__ uint64_t bars[2 * STAGES];
    __shared__ float s_new[kStepRows];                                      // the new key's scores
    __shared__ __align__(16) float v_new[DV];
    __shared__ float2 part_ml[kStepRows];
    __shared__ int s_failed;
    float* part = reinterpret_cast<float*>(step_smem + Sh::OFF_PART);
    uint64_t *full = bars, *empty = bars + STAGES;
    const GroupedDims& d = a.d;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int split = blockIdx.x, splits = gridDim.x, b = blockIdx.z;
    const int kvh = blockIdx.y / row_tiles, row0 = blockIdx.y % row_tiles * kStepRows, group = d.group();
    const int rows = min(group - row0, kStepRows);
    if (threadIdx.x == 0) {
        s_failed = 0;
        for (int s = 0; s < STAGES; ++s) { dme::mbar_init(&full[s], 1); dme::mbar_init(&empty[s], kStepWarps); }
        dme::mbar_init_fence();
    }
    __syncthreads();
    // the position was written by a launch that had completed before the step's first kernel began
    const int pos = a.pos_dev ? min(*a.pos_dev, a.max_seq - 1) : a.pos0;
    const int first = a.mask.first(pos);
    const int per = ((pos - first + splits - 1) / splits + 15) / 16 * 16;   // cached keys per CTA
    const int k0 = min(first + split * per, pos), k1 = min(k0 + per, pos);
    const int ntiles = (k1 - k0 + kStepKeys - 1) / kStepKeys;

    if (warp == kStepWarps) {
        if (lane == 0) {
            dme::prefetch_tensor_map(&mapK); dme::prefetch_tensor_map(&mapV);
            dme::Ring<STAGES> ring;
            for (int t = 0; t < ntiles; ++t) {
                if (t >= STAGES && !dme::wait(&empty[ring.stage], ring.phase ^ 1u, a.abort_word)) { atomicExch(&s_failed, 1); break; }
                unsigned char* dst = step_smem + ring.stage * Sh::STAGE;
                dme::mbar_arrive_expect_tx(&full[ring.stage], Sh::STAGE);
                #pragma unroll
                for (int x = 0; x < QKS; ++x) dme::copy_tile_4d(dst + x * Sh::BOX, &mapK, x * 64, k0 + t * kStepKeys, kvh, b, &full[ring.stage]);
                #pragma unroll
                for (int x = 0; x < VS; ++x) dme::copy_tile_4d(dst + (QKS + x) * Sh::BOX, &mapV, x * 64, k0 + t * kStepKeys, kvh, b, &full[ring.stage]);
                ring.advance();
            }
        }
        __syncwarp();
        griddep_wait();
    } else {
        griddep_wait();
        auto sync = [] { asm volatile("bar.sync 1, %0;" :: "n"(kStepThreads) : "memory"); };
        const int g = lane / 4, t4 = lane % 4, mi = lane / 8, r8 = lane % 8;
        const float scale_log2 = a.scale * kLog2e;
        // ---- the new key and value, the query rows ----------------------------------------------------------
        const float* p = static_cast<const float*>(a.proj) + size_t(b) * d.proj_row();
        const int col = 4 * lane;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        auto round4 = [](const float4& v) { return make_float4(to_float(from_float<T16>(v.x)), to_float(from_float<T16>(v.y)), to_float(from_float<T16>(v.z)), to_float(from_float<T16>(v.w))); };
        auto head = [&](const float4& raw) {                                // rotated, normalised, as the cache holds it
            const float f = a.norm ? rsqrtf(wave::dpp::reduce_sum(dot4(raw, raw)) / d.n_dim + a.eps) : 1.f;
            return round4(scaled(a.cos_t && col < d.dim ? rotate_quad(raw, a, pos, col) : raw, f));
        };
        const float4 k_raw = col < d.dim ? load4<float>(p + d.k_col() + size_t(kvh) * d.dim + col) : zero;
        float4 q_raw[2];
        #pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int r = warp + kStepWarps * i;
            q_raw[i] = r < rows && col < d.dim ? load4<float>(p + (size_t(kvh) * group + row0 + r) * d.dim + col) : zero;
        }
        const float4 kn = head(k_raw);
        unsigned char* qs = step_smem + Sh::OFF_Q;
        #pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int r = warp + kStepWarps * i;
            const float4 qn = head(q_raw[i]);
            if (col < 64 * QKS)
                *reinterpret_cast<uint2*>(qs + (col >> 6) * (kStepRows * 128) + swz128(r, (col & 63) >> 3) + (col & 4) * 2) = make_uint2(pack2<T16>(qn.x, qn.y), pack2<T16>(qn.z, qn.w));
            const float s = wave::dpp::reduce_sum(dot4(qn, kn));
            if (lane == 0) s_new[r] = s * scale_log2;
        }
        if (split == 0 && warp == 0) {
            const float4 v = round4(!d.own_values ? k_raw : col < d.vdim ? load4<float>(p + d.v_col() + size_t(kvh) * d.vdim + col) : zero);
            if (col < DV) store4<float>(v_new + col, v);
            if (row0 == 0) {
                const size_t at = (size_t(b) * d.kv_heads + kvh) * a.max_seq + pos;
                if (col < d.dim) store4<T16>(static_cast<T16*>(a.kcache) + at * d.dim + col, kn);
                if (col < d.vdim) store4<T16>(static_cast<T16*>(a.vcache) + at * d.vdim + col, v);
            }
        }
        sync();
        uint32_t qa[KS][4];
        #pragma unroll
        for (int ks = 0; ks < KS; ++ks)
            ldmatrix_x4(qa[ks], dme::smem_addr(qs) + (ks >> 2) * (kStepRows * 128) + swz128((mi & 1) * 8 + r8, 2 * (ks & 3) + (mi >> 1)));
        // ---- the cached keys --------------------------------------------------------------------------------
        float o[DV / 8][4];
        #pragma unroll
        for (int n = 0; n < DV / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
        float m0 = kNegBig, m1 = kNegBig, l0 = 0.f, l1 = 0.f;
        const int krow = warp * 16 + (mi >> 1) * 8 + r8, kchunk = mi & 1, vrow = warp * 16 + (mi & 1) * 8 + r8, vchunk = mi >> 1;
        dme::Ring<STAGES> ring;
        for (int t = 0; t < ntiles; ++t) {
            bool ok = dme::wait(&full[ring.stage], ring.phase, a.abort_word);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) { if (lane == 0) atomicExch(&s_failed, 1); break; }
            const uint32_t kt = dme::smem_addr(step_smem + ring.stage * Sh::STAGE), vt = kt + QKS * Sh::BOX;
            float s[4][4];                                                  // [n-tile + 2 * (odd k-step)]
            #pragma unroll
            for (int x = 0; x < 4; ++x) s[x][0] = s[x][1] = s[x][2] = s[x][3] = 0.f;
            #pragma unroll
            for (int ks = 0; ks < KS; ++ks) {
                const int cc = 2 * ks + kchunk;
                uint32_t bk[4];
                ldmatrix_x4(bk, kt + (cc >> 3) * Sh::BOX + swz128(krow, cc & 7));
                mma_16816<T16>(s[2 * (ks & 1)], qa[ks], bk[0], bk[1]);
                mma_16816<T16>(s[2 * (ks & 1) + 1], qa[ks], bk[2], bk[3]);
            }
            const int key = k0 + t * kStepKeys + warp * 16 + 2 * t4;
            float sc[2][4];
            #pragma unroll
            for (int n = 0; n < 2; ++n)
                #pragma unroll
                for (int j = 0; j < 4; ++j) sc[n][j] = key + n * 8 + (j & 1) < k1 ? (s[n][j] + s[2 + n][j]) * scale_log2 : kNegBig;
            const float n0 = fmaxf(m0, wave::lane_group_reduce<4>(fmaxf(fmaxf(sc[0][0], sc[0][1]), fmaxf(sc[1][0], sc[1][1])), wave::MaxOp{}));
            const float n1 = fmaxf(m1, wave::lane_group_reduce<4>(fmaxf(fmaxf(sc[0][2], sc[0][3]), fmaxf(sc[1][2], sc[1][3])), wave::MaxOp{}));
            if (__any_sync(0xffffffffu, n0 != m0 || n1 != m1)) {
                const float f0 = fast_exp2(m0 - n0), f1 = fast_exp2(m1 - n1);
                l0 *= f0; l1 *= f1;
                #pragma unroll
                for (int n = 0; n < DV / 8; ++n) { o[n][0] *= f0; o[n][1] *= f0; o[n][2] *= f1; o[n][3] *= f1; }
                m0 = n0; m1 = n1;
            }
            float pr[2][4];
            #pragma unroll
            for (int n = 0; n < 2; ++n) {
                #pragma unroll
                for (int j = 0; j < 4; ++j) pr[n][j] = sc[n][j] > kNegBig ? fast_exp2(sc[n][j] - (j < 2 ? m0 : m1)) : 0.f;
                l0 += pr[n][0] + pr[n][1];
                l1 += pr[n][2] + pr[n][3];
            }
            const uint32_t pa[4] = {pack2<T16>(pr[0][0], pr[0][1]), pack2<T16>(pr[0][2], pr[0][3]), pack2<T16>(pr[1][0], pr[1][1]), pack2<T16>(pr[1][2], pr[1][3])};
            #pragma unroll
            for (int n = 0; n < DV / 16; ++n) {
                const int cc = 2 * n + vchunk;
                uint32_t bv[4];
                ldmatrix_x4_trans(bv, vt + (cc >> 3) * Sh::BOX + swz128(vrow, cc & 7));
                mma_16816<T16>(o[2 * n], pa, bv[0], bv[1]);
                mma_16816<T16>(o[2 * n + 1], pa, bv[2], bv[3]);
            }
            __syncwarp();
            if (lane == 0) dme::mbar_arrive(&empty[ring.stage]);
            ring.advance();
        }
        l0 = wave::lane_group_reduce<4>(l0, wave::SumOp{});
        l1 = wave::lane_group_reduce<4>(l1, wave::SumOp{});
        // ---- the warps' results, the new key and the extra term meet (the ring is dead past this barrier) ---------
        sync();
        float* sm_o = reinterpret_cast<float*>(step_smem);                  // [warp][16][DP]
        float2* sm_ml = reinterpret_cast<float2*>(sm_o + kStepWarps * kStepRows * DP);
        #pragma unroll
        for (int n = 0; n < DV / 8; ++n) {
            *reinterpret_cast<float2*>(&sm_o[(warp * 16 + g) * DP + n * 8 + 2 * t4]) = make_float2(o[n][0], o[n][1]);
            *reinterpret_cast<float2*>(&sm_o[(warp * 16 + g + 8) * DP + n * 8 + 2 * t4]) = make_float2(o[n][2], o[n][3]);
        }
        if (t4 == 0) { sm_ml[warp * 16 + g] = make_float2(m0, l0); sm_ml[warp * 16 + g + 8] = make_float2(m1, l1); }
        sync();
        for (int e = 2 * threadIdx.x; e < rows * DV; e += 2 * kStepThreads) {
            const int r = e / DV, c = e % DV;
            float M = split == 0 ? fmaxf(s_new[r], a.plus_one ? 0.f : kNegBig) : kNegBig;
            #pragma unroll
            for (int w = 0; w < kStepWarps; ++w) M = fmaxf(M, sm_ml[w * 16 + r].x);
            float L = 0.f, o0 = 0.f, o1 = 0.f;
            if (split == 0) {
                const float f = fast_exp2(s_new[r] - M);
                L = f + (a.plus_one ? fast_exp2(-M) : 0.f);
                o0 = f * v_new[c]; o1 = f * v_new[c + 1];
            }
            #pragma unroll
            for (int w = 0; w < kStepWarps; ++w) {
                const float2 ml = sm_ml[w * 16 + r], ov = *reinterpret_cast<const float2*>(&sm_o[(w * 16 + r) * DP + c]);
                const float f = fast_exp2(ml.x - M);
                L += f * ml.y; o0 += f * ov.x; o1 += f * ov.y;
            }
            *reinterpret_cast<float2*>(&part[r * DV + c]) = make_float2(o0, o1);
            if (c == 0) part_ml[r] = make_float2(M, L);
        }
    }
    // ---- the CTAs' results meet; each finishes its share of the columns ------------------------------------------
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    const int total = rows * d.vdim / 2;
    for (int e = split * blockDim.x + threadIdx.x; e < total; e += splits * blockDim.x) {
        const int r = 2 * e / d.vdim, c = 2 * e % d.vdim;
        float M = kNegBig, L = 0.f, o0 = 0.f, o1 = 0.f;
        for (int s = 0; s < splits; ++s) M = fmaxf(M, cluster.map_shared_rank(part_ml, s)[r].x);
        for (int s = 0; s < splits; ++s) {
            const float2 ml = cluster.map_shared_rank(part_ml, s)[r];
            const float2 ov = *reinterpret_cast<const float2*>(cluster.map_shared_rank(part, s) + r * DV + c);
            const float f = fast_exp2(ml.x - M);
            L += f * ml.y; o0 += f * ov.x; o1 += f * ov.y;
        }
        float f0 = 1.f / L, f1 = f0;
        const size_t hcol = (size_t(kvh) * group + row0 + r) * d.vdim + c;
        if (d.gated) {
            const float2 gt = *reinterpret_cast<const float2*>(static_cast<const float*>(a.proj) + size_t(b) * d.proj_row() + d.g_col() + hcol);
            f0 /= 1.f + expf(-gt.x); f1 /= 1.f + expf(-gt.y);
        }
        *reinterpret_cast<uint32_t*>(static_cast<T16*>(a.out) + size_t(b) * d.v_row() + hcol) = pack2<T16>(o0 * f0, o1 * f1);
    }
    if (threadIdx.x == 0 && s_failed) { atomicExch(a.abort_word, 1); atomicExch(sticky, 1); }
    cluster.sync();                                                         // nobody leaves while its results are being read
}

template <int QKS, int VS>
int launch_step(const GroupedAttn& a, cudaStream_t st) {
    using Sh = StepSmem<QKS, VS>;
    const GroupedDims& d = a.d;
    CUtensorMap mk, mv;
    auto map = [&](CUtensorMap* m, const void* base, int cols) {
        const uint64_t row = uint64_t(cols) * 2, hd = row * a.max_seq;
        const uint64_t dims[4] = {uint64_t(cols), uint64_t(a.max_seq), uint64_t(d.kv_heads), uint64_t(a.batch)}, strides[3] = {row, hd, hd * d.kv_heads};
        const uint32_t box[4] = {64, kStepKeys, 1, 1};
        return make_tensor_map(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, base, dims, strides, box, Swizzle::B128);
    };
    cudaError_t e = map(&mk, a.kcache, d.dim);
    if (e == cudaSuccess) e = map(&mv, a.vcache, d.vdim);
    if (e != cudaSuccess) return int(e);
    int* sticky = device_status_ptr();
    if (!sticky) return B200P_E_NO_DEVICE;
    auto kern = grouped_step_kernel<QKS, VS>;
    if ((e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::BYTES))) return int(e);
    // splits: at least 256 keys each, no more CTAs than SMs, a cluster's worth; depends on nothing that changes from step to step
    const int row_tiles = (d.group() + kStepRows - 1) / kStepRows, sms = std::max(sm_count(), 1);
    const int keys = a.mask.kind == MASK_CAUSAL ? a.max_seq : std::min(a.mask.size, a.max_seq);
    int splits = 1;
    while (splits < 8 && keys > 256 * splits && 2 * splits * d.kv_heads * row_tiles * a.batch <= sms) splits *= 2;
    const int forced = tuning(KNOB_DECODE_SPLITS, 0);
    if (forced > 0) splits = std::min(forced, 8);
    return launch_dependent_clusters(kern, splits, dim3(unsigned(splits), unsigned(d.kv_heads * row_tiles), unsigned(a.batch)), kStepThreads + 32, Sh::BYTES, st,
                                     a, mk, mv, row_tiles, sticky);
}

} // namespace

int grouped_inputs(const GroupedAttn& a, cudaStream_t st) {
    if (a.d.dim > 512 || a.d.vdim > 512) return B200P_E_DIM;
    return a.dtype == B200P_F32 ? launch_inputs<float>(a, st) : launch_inputs<T16>(a, st);
}

int grouped_plain(const GroupedAttn& a, cudaStream_t st) {
    if (a.d.heads > 65535 || a.batch > 65535) return B200P_E_RANGE;
    return a.dtype == B200P_F32 ? launch_plain_t<float>(a, st) : launch_plain_t<T16>(a, st);
}

bool grouped_step_ok(const GroupedDims& d) { return d.dim <= 128 && d.vdim <= 128 && d.kv_heads * ((d.group() + kStepRows - 1) / kStepRows) <= 65535; }

int grouped_step(const GroupedAttn& a, cudaStream_t st) {
    const GroupedDims& d = a.d;
    if (a.dtype != B200P_BF16) return B200P_E_DTYPE;
    if (!grouped_step_ok(d) || a.Tn != 1 || a.batch > 65535) return B200P_E_RANGE;
    if (d.dim <= 64) return d.vdim <= 64 ? launch_step<1, 1>(a, st) : launch_step<1, 2>(a, st);
    return d.vdim <= 64 ? launch_step<2, 1>(a, st) : launch_step<2, 2>(a, st);
}

} // namespace b200p
