// Element-wise gate on the output of an attention kernel: out *= sigmoid(gate).
#pragma once
#include "attn_common.cuh"
#include "common.cuh"
#include "mma_sync.cuh"
#include "vec_quads.cuh"

namespace b200p {

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
    store8<T>(out + r * cols + c, x);
}

// rows x cols (a multiple of 8), rows of the gate gate_ld elements apart.
template <typename T, typename G>
int gate_rows(T* out, const G* gate, size_t rows, int cols, int gate_ld, cudaStream_t st) {
    const size_t n = rows * (cols / 8);
    gate_kernel<T, G><<<unsigned((n + 255) / 256), 256, 0, st>>>(out, gate, rows, cols, gate_ld);
    return launched();
}

} // namespace b200p
