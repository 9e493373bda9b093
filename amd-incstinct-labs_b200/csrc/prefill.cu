// ---------------------------------------------------------------------------
// prefill.cu -- the entry points of prefill attention (prefill_tc.cuh) for equal key
// and value head sizes of 64 and 128: cdna3::attn::prefill
// (cdna3-prims/include/cdna3/attention.hpp:86-109).
// ---------------------------------------------------------------------------
#include "prefill_tc.cuh"
#include "b200p.h"

namespace b200p {
namespace {

template <typename T, int D, int RS>
int launch_prefill_rs(const void* Q, const void* K, const void* V, void* O, const b200p_prefill_cfg* c, int dtype,
                   const b200p_attn_strides& s, float* debug_s, cudaStream_t st) {
    using Sh = PrefillShape<D>;
    const CUtensorMapDataType dt = dtype == B200P_F16 ? CU_TENSOR_MAP_DATA_TYPE_FLOAT16 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
    CUtensorMap mq, mk, mv;
    const uint64_t qd[4] = {uint64_t(D), uint64_t(c->seqQ), uint64_t(c->nQHeads), uint64_t(c->batch)};
    const uint64_t qs[3] = {uint64_t(s.q_seq) * 2, uint64_t(s.q_head) * 2, uint64_t(s.q_batch) * 2};
    const uint64_t kd[4] = {uint64_t(D), uint64_t(c->seqK), uint64_t(c->nKVHeads), uint64_t(c->batch)};
    const uint64_t ks[3] = {uint64_t(s.k_seq) * 2, uint64_t(s.k_head) * 2, uint64_t(s.k_batch) * 2};
    const uint64_t vs[3] = {uint64_t(s.v_seq) * 2, uint64_t(s.v_head) * 2, uint64_t(s.v_batch) * 2};
    const uint32_t box[4] = {64, 128, 1, 1};
    cudaError_t e = make_tensor_map(&mq, dt, 4, Q, qd, qs, box, Swizzle::B128);
    if (e == cudaSuccess) e = make_tensor_map(&mk, dt, 4, K, kd, ks, box, Swizzle::B128);
    if (e == cudaSuccess) e = make_tensor_map(&mv, dt, 4, V, kd, vs, box, Swizzle::B128);
    CUtensorMap mo;
    const uint64_t os[3] = {uint64_t(s.o_seq) * 2, uint64_t(s.o_head) * 2, uint64_t(s.o_batch) * 2};
    if (e == cudaSuccess) e = make_tensor_map(&mo, dt, 4, O, qd, os, box, Swizzle::B128);
    if (e != cudaSuccess) return int(e);

    const bool dbg = debug_s != nullptr;
    auto kern = dbg ? prefill_tc_kernel<T, Sh, RS, true> : prefill_tc_kernel<T, Sh, RS, false>;
    static bool attr_set[64][2] = {};
    int dev = 0; cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && !attr_set[dev][dbg]) {
        e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::SMEM_BYTES);
        if (e != cudaSuccess) return int(e);
        attr_set[dev][dbg] = true;
    }
    PrefillParams p{};
    p.debug_s = debug_s;
    p.sticky = device_status_ptr();
    LaunchSlot slot{};
    if (!p.sticky) return B200P_E_NO_DEVICE;
    if (int se = take_launch_slot(st, &slot)) return se;       // work counter and abort word of this launch, cleared on its stream
    p.status = slot.abort; p.work_counter = slot.work;
    p.seqQ = c->seqQ; p.seqK = c->seqK; p.nQH = c->nQHeads; p.nKVH = c->nKVHeads; p.group = c->nQHeads / c->nKVHeads;
    p.batch = c->batch; p.causal = c->causal;
    p.scale_log2 = 1.4426950408889634f / sqrtf(float(D));
    // One persistent CTA per SM (the kernel takes all of an SM's shared and tensor memory), or one CTA per
    // work item when the knob's bit 1 is set.
    const long long items = (long long)((c->seqQ + 2 * kBM - 1) / (2 * kBM)) * c->nQHeads * c->batch;
    if (items > 0x7fffffffLL / 2) return B200P_E_RANGE;
    const int sms = sm_count();
    const bool one_per_item = (tuning(KNOB_PREFILL_VARIANT, 0) & 2) != 0;
    dim3 grid(unsigned(one_per_item || items < sms ? items : sms), 1, 1);
    kern<<<grid, prefill_threads(RS), Sh::SMEM_BYTES, st>>>(p, mq, mk, mv, mo, mq, mk);
    return launched();
}

template <typename T, int D>
int launch_prefill(const void* Q, const void* K, const void* V, void* O, const b200p_prefill_cfg* c, int dtype,
                   const b200p_attn_strides& s, float* debug_s, cudaStream_t st) {
    return launch_prefill_rs<T, D, 1>(Q, K, V, O, c, dtype, s, debug_s, st);
}

} // namespace

int prefill_dispatch_strided(const void* Q, const void* K, const void* V, void* O, const b200p_prefill_cfg* c, int dtype,
                             const b200p_attn_strides* strides, float* debug_s, cudaStream_t st);

int prefill_dispatch(const void* Q, const void* K, const void* V, void* O, const b200p_prefill_cfg* c, int dtype,
                     float* debug_s, cudaStream_t st) {
    return prefill_dispatch_strided(Q, K, V, O, c, dtype, nullptr, debug_s, st);
}

int prefill_dispatch_strided(const void* Q, const void* K, const void* V, void* O, const b200p_prefill_cfg* c, int dtype,
                             const b200p_attn_strides* strides, float* debug_s, cudaStream_t st) {
    if (!c) return B200P_E_NULL;
    if (dtype != B200P_F16 && dtype != B200P_BF16) return B200P_E_DTYPE;
    if (c->D != 64 && c->D != 128) return B200P_E_DIM;                        // attention.hpp:105-107
    if (c->nQHeads <= 0 || c->nKVHeads <= 0 || c->nQHeads % c->nKVHeads != 0) return B200P_E_DIM;
    if (c->seqQ <= 0 || c->seqK <= 0 || c->batch <= 0) return B200P_E_LENGTH;
    if (c->nQHeads > 65535 || c->batch > 65535) return B200P_E_RANGE;
    if (!Q || !K || !V || !O) return B200P_E_NULL;
    if (!aligned(Q, 16) || !aligned(K, 16) || !aligned(V, 16) || !aligned(O, 16)) return B200P_E_ALIGN;
    if (sm_count() <= 0) return B200P_E_NO_DEVICE;
    b200p_attn_strides s;
    if (strides) {
        s = *strides;
        // TMA needs 16-byte multiples for every stride; the output rows are written with 16-byte stores
        const long long all[12] = {s.q_seq, s.q_head, s.q_batch, s.k_seq, s.k_head, s.k_batch,
                                   s.v_seq, s.v_head, s.v_batch, s.o_seq, s.o_head, s.o_batch};
        for (long long v : all) if (v <= 0 || (v * 2) % 16 != 0) return B200P_E_ALIGN;
    } else {                                                   // the reference's dense head-major layout
        const long long D = c->D;
        s.q_seq = D; s.q_head = (long long)c->seqQ * D; s.q_batch = (long long)c->nQHeads * c->seqQ * D;
        s.k_seq = D; s.k_head = (long long)c->seqK * D; s.k_batch = (long long)c->nKVHeads * c->seqK * D;
        s.v_seq = s.k_seq; s.v_head = s.k_head; s.v_batch = s.k_batch;
        s.o_seq = s.q_seq; s.o_head = s.q_head; s.o_batch = s.q_batch;
    }
    if (dtype == B200P_F16)
        return c->D == 128 ? launch_prefill<__half, 128>(Q, K, V, O, c, dtype, s, debug_s, st)
                           : launch_prefill<__half, 64>(Q, K, V, O, c, dtype, s, debug_s, st);
    return c->D == 128 ? launch_prefill<__nv_bfloat16, 128>(Q, K, V, O, c, dtype, s, debug_s, st)
                       : launch_prefill<__nv_bfloat16, 64>(Q, K, V, O, c, dtype, s, debug_s, st);
}

} // namespace b200p

using namespace b200p;

extern "C" int b200p_attn_prefill(const void* Q, const void* K, const void* V, void* O,
                                  const b200p_prefill_cfg* cfg, int dtype, b200p_stream_t stream) {
    return prefill_dispatch(Q, K, V, O, cfg, dtype, nullptr, static_cast<cudaStream_t>(stream));
}

extern "C" int b200p_attn_prefill_strided(const void* Q, const void* K, const void* V, void* O,
                                          const b200p_prefill_cfg* cfg, int dtype, const b200p_attn_strides* strides,
                                          b200p_stream_t stream) {
    if (!strides) return B200P_E_NULL;
    return prefill_dispatch_strided(Q, K, V, O, cfg, dtype, strides, nullptr, static_cast<cudaStream_t>(stream));
}

extern "C" int b200p_attn_prefill_debug(const void* Q, const void* K, const void* V, void* O,
                                        const b200p_prefill_cfg* cfg, int dtype, float* raw_scores,
                                        b200p_stream_t stream) {
    return prefill_dispatch(Q, K, V, O, cfg, dtype, raw_scores, static_cast<cudaStream_t>(stream));
}
