// ---------------------------------------------------------------------------
// latent.cuh -- latent attention: shapes, and the launchers of its kernels
// (latent_attn.cu: few query rows on the latent cache, and the plain kernel for any
// shape and type; latent_prefill.cu: tcgen05 prefill on expanded keys and values).
//
// Every position keeps ONE vector for all heads in the cache: a normalised latent
// of `rank` columns and a rotated key part of `rot` columns.  Per head the key is
// [W_uk latent | rotated part] and the value W_uv latent.  Two ways to attend:
//   expanded  W_uk, W_uv are applied to the cached latents (one GEMM over the
//             keys), then it is ordinary attention with a key part in common;
//   absorbed  W_uk^T is applied to the query instead, scores are taken against the
//             cached vector itself, the weighted latents are summed and W_uv is
//             applied to the sum: the cache is read once for all heads.
// All sizes here are padded to multiples of 16 with zero columns (the session packs
// the weights that way), so that every matrix and vector is tensor-core and TMA
// shaped whatever the model's sizes are.
// ---------------------------------------------------------------------------
#pragma once
#include <cuda_runtime.h>
#include "common.cuh"

namespace b200p {

struct LatentDims {
    int heads, dim, rot, vdim, rank, qrank;       // padded; rot holds whole groups of 8 pairs (see SkinnyPairRot)
    __host__ __device__ int cache_row() const { return rank + rot; }
    __host__ __device__ int q_row() const { return heads * (dim + rot); }
    __host__ __device__ int kv_row() const { return heads * (dim + vdim); }      // all heads' key parts, then all heads' values
    __host__ __device__ int v_row() const { return heads * vdim; }
    // the fused first projection: [query latent | latent | rotated key part | gate]
    __host__ __device__ int proj_row() const { return qrank + rank + rot + v_row(); }
    __host__ __device__ int gate_col() const { return qrank + rank + rot; }
};

// Attention of Tn new tokens per sequence (already in the cache) against all N = pos0 + Tn cached positions.
struct LatentAttn {
    LatentDims d;
    int dtype, batch, Tn, pos0, max_seq;
    float scale;
    const float* sink;             // [heads] or null: exp(sink) joins the softmax denominator
    const void* q;                 // [batch * Tn][q_row]: per head [plain | rotated]
    const void* kv;                // expanded: [batch][N][kv_row]
    const void* cache;             // [batch][max_seq][cache_row]
    const float* proj;             // [batch * Tn][proj_row]: the gate's pre-activations
    void* out;                     // [batch * Tn][v_row], gated
};

// A few new tokens per sequence (M = batch * Tn <= 16) on the latent cache: absorbed form, bf16, four launches.
struct LatentStep {
    LatentDims d;
    int batch, Tn, pos0, max_seq;
    const int* pos_dev;            // position of the first new token, read on the device (null: pos0)
    float scale, eps;
    int kv_rank;                   // columns of the latent without padding
    const float* sink;             // [heads] or null
    const void *ukT, *uv;          // [heads][rank][dim], [heads * vdim][rank]
    const void* kv_norm;           // [rank]
    const float *cos_t, *sin_t;    // [max_seq][rot / 2]
    const float* proj;             // [M][proj_row]
    const void* q_plain;           // [M][heads * dim]
    void* q_abs;                   // [M * heads][cache_row]: the rotated part is there already
    void* cache;                   // [batch][max_seq][cache_row]
    float *part_o, *part_ml;       // splits' partial results: latent_step_partials(d) rows of `rank` and of 2 floats
    void* merged;                  // [M * heads][rank]: weighted sums of the latents
    void* out;                     // [M][v_row], gated
    int* abort_word;
};
bool latent_step_ok(const LatentDims& d, int M);
size_t latent_step_partials(const LatentDims& d);
int latent_step_absorb(const LatentStep& a, cudaStream_t st);     // latents and rotated keys into the cache; W_uk^T q
int latent_step_attend(const LatentStep& a, cudaStream_t st);     // splits of the cache -> partial weighted latents
int latent_step_values(const LatentStep& a, cudaStream_t st);     // merge, W_uv, gate

// Any shape, bf16 or fp32 (fp32 arithmetic throughout).  Expanded form.
int latent_attn_plain(const LatentAttn& a, cudaStream_t st);
// tcgen05 (bf16; dim and vdim up to 128, rot up to 64; B200P_E_RANGE otherwise, nothing launched).  Expanded form.
int latent_attn_prefill(const LatentAttn& a, cudaStream_t st);

} // namespace b200p
