// Four or eight consecutive elements of any type as fp32.
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

// eight consecutive elements as fp32 and back; p is aligned to 16 bytes
template <typename G> __device__ __forceinline__ void load8(const G* p, float (&f)[8]) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const G* e = reinterpret_cast<const G*>(&v);
    #pragma unroll
    for (int k = 0; k < 8; ++k) f[k] = to_float(e[k]);
}
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&f)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

template <typename T> __device__ __forceinline__ void store8(T* p, const float (&f)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack2<T>(f[0], f[1]), pack2<T>(f[2], f[3]), pack2<T>(f[4], f[5]), pack2<T>(f[6], f[7]));
}
template <> __device__ __forceinline__ void store8<float>(float* p, const float (&f)[8]) {
    reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}

} // namespace b200p
