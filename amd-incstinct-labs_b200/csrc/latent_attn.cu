// ---------------------------------------------------------------------------
// latent_attn.cu -- latent attention on CUDA cores and warp MMAs (latent.cuh).
// ---------------------------------------------------------------------------
#include "latent.cuh"
#include "attn_common.cuh"
#include "mma_sync.cuh"
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

} // namespace

int latent_attn_plain(const LatentAttn& a, cudaStream_t st) {
    if (a.d.heads > 65535 || a.batch > 65535) return B200P_E_RANGE;
    return a.dtype == B200P_F32 ? launch_plain_t<float>(a, st) : launch_plain_t<__nv_bfloat16>(a, st);
}

} // namespace b200p
