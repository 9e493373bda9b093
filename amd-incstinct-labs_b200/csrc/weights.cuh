// ---------------------------------------------------------------------------
// weights.cuh -- what decoders built from config.json share when a session is made: reading
// numbers of the configuration, copying stored tensors into packed and padded matrices, and
// tables of rotary angles.
// ---------------------------------------------------------------------------
#pragma once
#include "session.cuh"
#include "model.hpp"
#include <algorithm>
#include <cmath>
#include <functional>
#include <string>

namespace b200p {

inline int pad16(int n) { return (n + 15) / 16 * 16; }

// ---- configuration --------------------------------------------------------------------------------
inline bool read_int(const Json* obj, const char* key, int* out, int least = 1) {
    const Json* v = obj ? obj->get(key) : nullptr;
    if (!v || !v->is_int() || v->num < least || v->num > 1e9) return false;
    *out = int(v->num);
    return true;
}
inline bool read_num(const Json* obj, const char* key, double* out) {
    const Json* v = obj ? obj->get(key) : nullptr;
    if (!v || v->kind != Json::Number) return false;
    *out = v->num;
    return true;
}

// ---- packed weights -------------------------------------------------------------------------------
// Element (r, c) of a stored matrix goes to dst[row_at[r] + col_at[c]].
template <typename T>
__global__ void pack_kernel(T* __restrict__ dst, const void* __restrict__ src, int src_dtype, int rows, int cols,
                            const long long* __restrict__ row_at, const long long* __restrict__ col_at) {
    const size_t n = size_t(rows) * cols;
    for (size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += size_t(gridDim.x) * blockDim.x) {
        const int r = int(i / cols), c = int(i % cols);
        const float v = src_dtype == B200P_BF16 ? to_float(static_cast<const __nv_bfloat16*>(src)[i])
                      : src_dtype == B200P_F16  ? to_float(static_cast<const __half*>(src)[i]) : static_cast<const float*>(src)[i];
        dst[row_at[r] + col_at[c]] = from_float<T>(v);
    }
}

// Where a row or a column of a stored tensor goes.
using Where = std::function<long long(int)>;
inline Where at_index() { return [](int i) -> long long { return i; }; }
inline Where at_stride(long long ld, long long first = 0) { return [=](int i) { return (first + i) * ld; }; }
// index i = head * n + j -> (head * np + j) * ld + first: heads of n entries, padded to np
inline Where at_heads(int n, int np, long long ld = 1, long long first = 0) {
    return [=](int i) { return (first + (long long)(i / n) * np + i % n) * ld; };
}

template <typename T> inline int type_code();
template <> inline int type_code<float>() { return B200P_F32; }
template <> inline int type_code<__nv_bfloat16>() { return B200P_BF16; }

template <typename T>
int pack(T* dst, const TensorRef& t, const Where& row_at, const Where& col_at) {
    const int rows = t.shape.size() > 1 ? int(t.shape[0]) : 1, cols = int(t.shape.back());
    if (t.dtype != B200P_BF16 && t.dtype != B200P_F16 && t.dtype != B200P_F32) return B200P_E_DTYPE;
    std::vector<long long> at(size_t(rows) + cols);
    for (int r = 0; r < rows; ++r) at[r] = row_at(r);
    for (int c = 0; c < cols; ++c) at[size_t(rows) + c] = col_at(c);
    long long* dev = nullptr;
    if (cudaError_t e = cudaMalloc(&dev, at.size() * sizeof(long long))) return int(e);
    cudaError_t e = cudaMemcpy(dev, at.data(), at.size() * sizeof(long long), cudaMemcpyHostToDevice);
    if (e == cudaSuccess) {
        const size_t n = size_t(rows) * cols;
        pack_kernel<T><<<unsigned(std::min<size_t>((n + 255) / 256, 8192)), 256>>>(dst, t.dev, t.dtype, rows, cols, dev, dev + rows);
        const int rc = launched();
        e = rc ? cudaError_t(rc) : cudaDeviceSynchronize();
    }
    cudaFree(dev);
    return int(e);
}

// Packs a model's tensors into memory of the session, elements of type T; the first error stays in rc and stops the rest.
template <typename T> struct WeightPacker {
    b200p_session* s;
    const b200p_model* m;
    int rc = B200P_OK;

    void* zeros(size_t n, size_t esz) {
        void* p = nullptr;
        if (rc) return nullptr;
        if (cudaError_t e = s->alloc(&p, n * esz)) { rc = int(e); return nullptr; }
        if (cudaError_t e = cudaMemset(p, 0, n * esz)) { rc = int(e); return nullptr; }
        return p;
    }
    void put(void* dst, const std::string& name, const Where& row_at, const Where& col_at) {
        if (!rc) rc = pack<T>(static_cast<T*>(dst), m->tensors.at(name), row_at, col_at);
    }
    void put_f32(float* dst, const std::string& name, const Where& row_at, const Where& col_at) {
        if (!rc) rc = pack<float>(dst, m->tensors.at(name), row_at, col_at);
    }
    // a whole matrix or vector whose rows only need padding to `ld` columns (and `rows_p` rows); as it is when they need none
    void* padded(const std::string& name, int rows_p, int ld) {
        const TensorRef& t = m->tensors.at(name);
        const int rows = t.shape.size() > 1 ? int(t.shape[0]) : 1;
        if (t.dtype == type_code<T>() && rows == rows_p && t.shape.back() == ld && aligned(t.dev, 32)) return const_cast<void*>(t.dev);
        void* p = zeros(size_t(rows_p) * ld, sizeof(T));
        put(p, name, at_stride(ld), at_index());
        return p;
    }
};

// cos and sin of p * freq[i], [max_seq][pairs]; pairs past the frequencies do not turn.  Angles in double.
inline int rotation_table(b200p_session* s, const std::vector<double>& freq, int pairs, std::pair<float*, float*>* out) {
    std::vector<float> c(size_t(s->max_seq) * pairs, 1.f), sn(c.size(), 0.f);
    for (size_t i = 0; i < freq.size(); ++i)
        for (int p = 0; p < s->max_seq; ++p) {
            c[size_t(p) * pairs + i] = float(std::cos(p * freq[i]));
            sn[size_t(p) * pairs + i] = float(std::sin(p * freq[i]));
        }
    cudaError_t e;
    if ((e = s->alloc(&out->first, c.size() * 4)) || (e = s->alloc(&out->second, c.size() * 4))) return int(e);
    if ((e = cudaMemcpy(out->first, c.data(), c.size() * 4, cudaMemcpyHostToDevice))) return int(e);
    return int(cudaMemcpy(out->second, sn.data(), c.size() * 4, cudaMemcpyHostToDevice));
}

} // namespace b200p
