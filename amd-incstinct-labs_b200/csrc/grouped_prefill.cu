// ---------------------------------------------------------------------------
// grouped_prefill.cu -- grouped attention over many new tokens: the tcgen05 prefill kernel
// (prefill_tc.cuh) on the cache, with a mask's first key, a causal offset for portions of
// prompts and keys and values of different widths; then the gate.
// ---------------------------------------------------------------------------
#include "grouped_attn.cuh"
#include "gate_rows.cuh"
#include "prefill_tc.cuh"
#include "b200p.h"

namespace b200p {
namespace {

template <typename T, int QKS, int VS>
int launch(const GroupedAttn& a, cudaStream_t st) {
    using Sh = MaskedPrefillShape<QKS, VS>;
    const GroupedDims& d = a.d;
    const int N = a.pos0 + a.Tn;
    CUtensorMap mq, mk, mv, mo;
    auto map = [&](CUtensorMap* m, const void* base, int cols, int rows, int heads, long long row, long long head, long long seq) {
        const uint64_t dims[4] = {uint64_t(cols), uint64_t(rows), uint64_t(heads), uint64_t(a.batch)};
        const uint64_t strides[3] = {uint64_t(row) * 2, uint64_t(head) * 2, uint64_t(seq) * 2};
        const uint32_t box[4] = {64, 128, 1, 1};
        return make_tensor_map(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, base, dims, strides, box, Swizzle::B128);
    };
    const long long qrow = d.proj_row(), vrow = d.v_row(), khead = (long long)a.max_seq * d.dim, vhead = (long long)a.max_seq * d.vdim;
    cudaError_t e = map(&mq, a.proj, d.dim, a.Tn, d.heads, qrow, d.dim, a.Tn * qrow);
    if (e == cudaSuccess) e = map(&mk, a.kcache, d.dim, N, d.kv_heads, d.dim, khead, d.kv_heads * khead);
    if (e == cudaSuccess) e = map(&mv, a.vcache, d.vdim, N, d.kv_heads, d.vdim, vhead, d.kv_heads * vhead);
    if (e == cudaSuccess) e = map(&mo, a.out, d.vdim, a.Tn, d.heads, vrow, d.vdim, a.Tn * vrow);
    if (e != cudaSuccess) return int(e);
    auto kern = prefill_tc_kernel<T, Sh, 1, false>;
    if ((e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::SMEM_BYTES))) return int(e);
    PrefillParams p{};
    p.sticky = device_status_ptr();
    if (!p.sticky) return B200P_E_NO_DEVICE;
    const long long items = (long long)((a.Tn + 2 * kBM - 1) / (2 * kBM)) * d.heads * a.batch;
    if (items > 0x7fffffffLL / 2) return B200P_E_RANGE;
    LaunchSlot slot{};
    if (int se = take_launch_slot(st, &slot)) return se;
    p.status = slot.abort; p.work_counter = slot.work;
    p.seqQ = a.Tn; p.seqK = N; p.nQH = d.heads; p.nKVH = d.kv_heads; p.group = d.group(); p.batch = a.batch; p.causal = 1;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.pos0 = a.pos0; p.v_cols = d.vdim; p.mask = a.mask; p.plus_one = a.plus_one ? 1 : 0;
    const int sms = sm_count();
    kern<<<unsigned(items < sms ? items : sms), prefill_threads(1), Sh::SMEM_BYTES, st>>>(p, mq, mk, mv, mo, mq, mk);
    if (int le = launched()) return le;
    if (!d.gated) return B200P_OK;
    return gate_rows(static_cast<T*>(a.out), static_cast<const T*>(a.proj) + d.g_col(), size_t(a.batch) * a.Tn, int(vrow), d.proj_row(), st);
}

} // namespace

int grouped_prefill(const GroupedAttn& a, cudaStream_t st) {
    const GroupedDims& d = a.d;
    if (a.dtype != B200P_BF16) return B200P_E_DTYPE;
    if (d.dim > 128 || d.vdim > 128 || d.heads > 65535 || a.batch > 65535) return B200P_E_RANGE;
    using T = __nv_bfloat16;
    if (d.dim <= 64) return d.vdim <= 64 ? launch<T, 1, 1>(a, st) : launch<T, 1, 2>(a, st);
    return d.vdim <= 64 ? launch<T, 2, 1>(a, st) : launch<T, 2, 2>(a, st);
}

} // namespace b200p
