// ---------------------------------------------------------------------------
// delta.cuh -- the gated delta rule: a layer whose memory of a sequence is one matrix S
// [dim][vdim] per head (and the last inputs of short convolutions), carried in fp32.
//
// Per token and head, with unit vectors k and q (q also by dim^-1/2), a decay g and a step beta:
//     S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q
// q, k and v come out of a projection through a causal convolution per channel and silu; o is
// divided by its root mean square over vdim, scaled by a weight and gated by silu.
//
// Many tokens go in blocks of sixteen.  With G_t the product of the block's decays up to t, R_it that of
// the decays between i and t (products of decays, never a quotient) and S0 the state ahead of the block,
//     u_t = beta_t (v_t - G_t S0^T k_t - sum_{i<t} R_it (k_i.k_t) u_i)
//     o_t = G_t S0^T q_t + sum_{i<=t} R_it (k_i.q_t) u_i
// Solving the triangle for u (T = (1 + L)^-1 diag(beta), L_ti = beta_t R_it k_i.k_t) and putting it into
// o (M_ti = R_it k_i.q_t) leaves everything that depends on the block alone to be computed for all blocks
// at once, and a step from block to block without a triangle:
//     u = T V - (T G K) S0,   o = M T V + (G Q - M T G K) S0,   S = G_16 S0 + sum_i R_i16 k_i u_i^T
// The state, decays, steps and unit vectors are fp32; products keep fp32 accuracy (delta_rule.cu).
//
// Sizes are padded with zero columns: dim and vdim to multiples of 16 in the projection, the
// rows of S to a multiple of 32.
// ---------------------------------------------------------------------------
#pragma once
#include <cuda_runtime.h>
#include "common.cuh"

namespace b200p {

struct DeltaDims {
    int heads, kv_heads;           // head h uses query/key head h / (heads / kv_heads)
    int dim, vdim;                 // padded to multiples of 16
    int n_dim, n_vdim;             // without padding
    int taps;                      // of the convolutions, the current token's included
    __host__ __device__ int group() const { return heads / kv_heads; }
    __host__ __device__ int rows() const { return (dim + 31) / 32 * 32; }                  // of S
    __host__ __device__ int channels() const { return 2 * kv_heads * dim + heads * vdim; } // with a convolution: [q | k | v]
    __host__ __device__ int g_col() const { return channels(); }
    __host__ __device__ int v_row() const { return heads * vdim; }
    __host__ __device__ int main_row() const { return channels() + heads * vdim; }         // [q | k | v | gate]
    __host__ __device__ int ab_row() const { return (2 * heads + 15) / 16 * 16; }          // [decay inputs | step inputs], always fp32
    __host__ __device__ size_t state_floats() const { return size_t(heads) * rows() * vdim; }
    // one block of sixteen tokens of a head: [16][rows] of T G K, of G Q - M T G K and of R_i16 k_i, then G_16
    // (tensor-core form: the first two with rows 16 longer, the third as [rows][16])
    __host__ __device__ int row_block(bool tensor) const { return 48 * rows() + 4 + (tensor ? 512 : 0); }
};
constexpr int kDeltaBlock = 16;

struct DeltaArgs {
    DeltaDims d;
    int dtype, batch, Tn, pos0, max_seq;
    const int* pos_dev;            // delta_step: the new token's position, read on the device (null: pos0)
    float eps;
    const void* proj;              // [batch * Tn][ldp]: columns [q | k | v | gate]
    int ldp, proj_dtype;
    const float* ab;               // [batch * Tn][ld_ab]
    int ld_ab;
    const float* conv;             // [taps][channels]; the last row is the current token's
    const float *a_log, *dt_bias;  // [heads]
    const float* norm;             // [vdim]
    float* state;                  // [batch][heads][rows][vdim]; position 0 starts from zero whatever it holds
    float* ring;                   // [batch][taps][channels]: the convolutions' input at position p is in slot p % taps
    // many tokens only: blocks = ceil(Tn / 16)
    float* rows;                   // [batch][heads][blocks][row_block]
    float* cols;                   // [batch][heads][vdim / 16][blocks][2][16 tokens][16 columns]: T V, M T V (tensor-core form: columns x tokens)
    float* o;                      // [batch * Tn][v_row]
    void* out;                     // [batch * Tn][v_row]: normalised and gated, of type dtype
    int* abort_word;
};

// Any number of new tokens.  bf16 or fp32; dim up to 512.
int delta_tokens(const DeltaArgs& a, cudaStream_t st);
// One new token per sequence, one launch.
bool delta_step_ok(const DeltaDims& d);
int delta_step(const DeltaArgs& a, cudaStream_t st);

// Floats of the buffers for up to M tokens of all sequences.
struct DeltaScratch { size_t rows, cols, o; };
inline DeltaScratch delta_scratch(const DeltaDims& d, int batch, int M) {
    const size_t blocks = (size_t(M) + size_t(batch) * (kDeltaBlock - 1)) / kDeltaBlock;        // every sequence may end in a partial one
    return {blocks * d.heads * d.row_block(true), blocks * d.heads * d.vdim * 32, size_t(M) * d.v_row()};
}

} // namespace b200p
