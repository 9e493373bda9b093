// ---------------------------------------------------------------------------
// grouped_attn.cuh -- attention of grouped query heads under a mask that bounds how far back a
// query sees (AttnMask: window, chunk or nothing): shapes and launchers.
//
// What varies between models are parameters: rotary positions on the first dimensions of query
// and key (adjacent pairs), a weightless RMS norm of both per head, values of their own or the
// keys as projected, one more term in the softmax's denominator, a sigmoid gate on the output.
// Head sizes are padded to multiples of 16 with zero columns (the session packs the weights
// that way), so every row is TMA shaped whatever the model's sizes are.
//
//   grouped_inputs   a projection's rows: queries turned and normalised in place, keys and values into the cache
//   grouped_plain    any shape and type, fp32 arithmetic
//   grouped_prefill  many query rows: the tcgen05 kernel (prefill_tc.cuh)
//   grouped_step     one new token per sequence: one launch from the projection's fp32 rows to the
//                    gated output, the new key and value into the cache on the way
// ---------------------------------------------------------------------------
#pragma once
#include <cuda_runtime.h>
#include "attn_common.cuh"
#include "common.cuh"

namespace b200p {

struct GroupedDims {
    int heads, kv_heads;           // query head h reads key/value head h / (heads / kv_heads)
    int dim, vdim;                 // padded
    int n_dim;                     // query/key columns without padding: what the norm's mean is over
    bool own_values, gated;        // values of their own / the keys as projected; output gate
    __host__ __device__ int group() const { return heads / kv_heads; }
    __host__ __device__ int v_row() const { return heads * vdim; }
    // the projection: [queries | keys | values of their own | gate]
    __host__ __device__ int k_col() const { return heads * dim; }
    __host__ __device__ int v_col() const { return own_values ? k_col() + kv_heads * dim : k_col(); }
    __host__ __device__ int g_col() const { return k_col() + kv_heads * (dim + (own_values ? vdim : 0)); }
    __host__ __device__ int proj_row() const { return g_col() + (gated ? heads * vdim : 0); }
};

// New tokens pos0 .. pos0 + Tn - 1 of `batch` sequences.
struct GroupedAttn {
    GroupedDims d;
    AttnMask mask;
    int dtype, batch, Tn, pos0, max_seq;
    const int* pos_dev;            // grouped_step: the new token's position, read on the device (null: pos0)
    float scale, eps;
    bool norm, plus_one;           // queries and keys by their root mean square; e^0 joins the denominator
    const float *cos_t, *sin_t;    // [max_seq][dim / 2] (1 and 0 where nothing turns), or null: no positions
    const void* proj;              // [batch * Tn][proj_row]: the session's type; grouped_step: fp32.  grouped_inputs leaves the queries in it
    void *kcache, *vcache;         // [batch][kv_heads][max_seq][dim], [..][vdim]
    void* out;                     // [batch * Tn][v_row]
    int* abort_word;               // grouped_step: raised by a wait that gives up
};

int grouped_inputs(const GroupedAttn& a, cudaStream_t st);
int grouped_plain(const GroupedAttn& a, cudaStream_t st);
// bf16, dim and vdim up to 128; B200P_E_RANGE otherwise, nothing launched.  Without the gate.
int grouped_prefill(const GroupedAttn& a, cudaStream_t st);
// bf16, dim and vdim up to 128.
bool grouped_step_ok(const GroupedDims& d);
int grouped_step(const GroupedAttn& a, cudaStream_t st);

} // namespace b200p
