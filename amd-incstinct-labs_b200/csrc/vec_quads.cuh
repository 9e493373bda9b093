// Four consecutive elements of any type as fp32.
#pragma once
#include "attn_common.cuh"
#include "mma_sync.cuh"

namespace b200p {

// four elements as fp32 and back; p is aligned to four elements
template <typename T> __device__ __forceinline__ float4 load4(const T* p) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const T* e = reinterpret_cast<const T*>(&r);
    return make_float4(to_float(e[0]), to_float(e[1]), to_float(e[2]), to_float(e[3]));
}
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <typename T> __device__ __forceinline__ void store4(T* p, const float4& v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack2<T>(v.x, v.y), pack2<T>(v.z, v.w));
}
template <> __device__ __forceinline__ void store4<float>(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }

} // namespace b200p
