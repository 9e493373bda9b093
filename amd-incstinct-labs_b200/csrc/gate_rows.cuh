// Element-wise gate on the output of an attention kernel: out *= sigmoid(gate).
#pragma once
#include "attn_common.cuh"
#include "common.cuh"
#include "mma_sync.cuh"

namespace b200p {

// eight consecutive elements, 16-byte aligned, as fp32
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

// Eight columns per thread; T is a 16-bit type.
template <typename T, typename G>
__global__ void __launch_bounds__(256) gate_kernel(T* __restrict__ out, const G* __restrict__ gate, size_t rows, int cols, int gate_ld) {
    const size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x;
    const int per_row = cols / 8;
    if (i >= rows * per_row) return;
    const size_t r = i / per_row;
    const int c = int(i % per_row) * 8;
    float x[8], g[8];
    load8<T>(out + r * cols + c, x);
    load8<G>(gate + r * gate_ld + c, g);
    #pragma unroll
    for (int k = 0; k < 8; ++k) x[k] /= 1.f + __expf(-g[k]);
    *reinterpret_cast<uint4*>(out + r * cols + c) = make_uint4(pack2<T>(x[0], x[1]), pack2<T>(x[2], x[3]), pack2<T>(x[4], x[5]), pack2<T>(x[6], x[7]));
}

// rows x cols (a multiple of 8), rows of the gate gate_ld elements apart.
template <typename T, typename G>
int gate_rows(T* out, const G* gate, size_t rows, int cols, int gate_ld, cudaStream_t st) {
    const size_t n = rows * (cols / 8);
    gate_kernel<T, G><<<unsigned((n + 255) / 256), 256, 0, st>>>(out, gate, rows, cols, gate_ld);
    return launched();
}

} // namespace b200p
