// ---------------------------------------------------------------------------
// latent_prefill.cu -- latent attention over many new tokens: the tcgen05 prefill kernel
// (prefill_tc.cuh) on expanded keys and values (latent.cuh), and the gate.
// ---------------------------------------------------------------------------
#include "latent.cuh"
#include "prefill_tc.cuh"
#include "gate_rows.cuh"
#include "b200p.h"

namespace b200p {
namespace {

template <typename T, int PLAIN, int VS>
int launch(const LatentAttn& a, cudaStream_t st) {
    using Sh = LatentPrefillShape<PLAIN, VS>;
    const LatentDims& d = a.d;
    const int N = a.pos0 + a.Tn;
    const CUtensorMapDataType dt = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
    CUtensorMap mq, mk, mv, mo, mqr, mkr;
    auto map = [&](CUtensorMap* m, const void* base, int first, int cols, int rows, int heads, long long row, long long head, long long seq,
                   int box_cols, Swizzle sw) {
        const uint64_t dims[4] = {uint64_t(cols), uint64_t(rows), uint64_t(heads), uint64_t(a.batch)};
        const uint64_t strides[3] = {uint64_t(row) * 2, uint64_t(head) * 2, uint64_t(seq) * 2};
        const uint32_t box[4] = {uint32_t(box_cols), 128, 1, 1};
        return make_tensor_map(m, dt, 4, static_cast<const T*>(base) + first, dims, strides, box, sw);
    };
    const long long qrow = d.q_row(), krow = d.kv_row(), vrow = d.v_row(), crow = d.cache_row(), qh = d.dim + d.rot;
    cudaError_t e = map(&mq, a.q, 0, d.dim, a.Tn, d.heads, qrow, qh, a.Tn * qrow, 64, Swizzle::B128);
    if (e == cudaSuccess) e = map(&mqr, a.q, d.dim, d.rot, a.Tn, d.heads, qrow, qh, a.Tn * qrow, 64, Swizzle::B128);
    if (e == cudaSuccess) e = map(&mk, a.kv, 0, d.dim, N, d.heads, krow, d.dim, N * krow, 64, Swizzle::B128);
    if (e == cudaSuccess) e = map(&mkr, a.cache, d.rank, d.rot, N, 1, crow, crow, a.max_seq * crow, 64, Swizzle::B128);
    if (e == cudaSuccess) e = map(&mv, a.kv, d.heads * d.dim, d.vdim, N, d.heads, krow, d.vdim, N * krow, 64, Swizzle::B128);
    if (e == cudaSuccess) e = map(&mo, a.out, 0, d.vdim, a.Tn, d.heads, vrow, d.vdim, a.Tn * vrow, Sh::OUT_COLS, Swizzle::B64);
    if (e != cudaSuccess) return int(e);
    auto kern = prefill_tc_kernel<T, Sh, 1, false>;
    if ((e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::SMEM_BYTES))) return int(e);
    PrefillParams p{};
    p.sticky = device_status_ptr();
    if (!p.sticky) return B200P_E_NO_DEVICE;
    LaunchSlot slot{};
    if (int se = take_launch_slot(st, &slot)) return se;
    p.status = slot.abort; p.work_counter = slot.work;
    p.seqQ = a.Tn; p.seqK = N; p.nQH = p.nKVH = d.heads; p.group = 1; p.batch = a.batch; p.causal = 1;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.pos0 = a.pos0; p.v_cols = d.vdim; p.sink = a.sink;
    const long long items = (long long)((a.Tn + 2 * kBM - 1) / (2 * kBM)) * d.heads * a.batch;
    if (items > 0x7fffffffLL / 2) return B200P_E_RANGE;
    const int sms = sm_count();
    kern<<<unsigned(items < sms ? items : sms), prefill_threads(1), Sh::SMEM_BYTES, st>>>(p, mq, mk, mv, mo, mqr, mkr);
    if (int le = launched()) return le;
    return gate_rows(static_cast<T*>(a.out), a.proj + d.gate_col(), size_t(a.batch) * a.Tn, int(vrow), d.proj_row(), st);
}

} // namespace

int latent_attn_prefill(const LatentAttn& a, cudaStream_t st) {
    const LatentDims& d = a.d;
    if (a.dtype != B200P_BF16) return B200P_E_DTYPE;
    if (d.dim > 128 || d.rot > 64 || d.vdim > 128 || d.heads > 65535 || a.batch > 65535) return B200P_E_RANGE;
    using T = __nv_bfloat16;
    if (d.dim <= 64) return d.vdim <= 64 ? launch<T, 1, 1>(a, st) : launch<T, 1, 2>(a, st);
    return d.vdim <= 64 ? launch<T, 2, 1>(a, st) : launch<T, 2, 2>(a, st);
}

} // namespace b200p
