// The walk over a matrix memory (linear_attention.cu) as the other kernels' host code sees it.
#pragma once

#include "common.cuh"

namespace mlc {

// S_t = diag(a_t) S_{t-1} + k_t v_tᵀ,  o_t = S_tᵀ (q_t · q_scale)  per sequence and head, S [dim][vdim]
struct GlaArgs {
    const float* qk;            // rows that hold q (at q_col) and k (at k_col)
    long long qk_stride;
    const float* vsrc;          // rows that hold v (at v_col); may be the same matrix
    long long v_stride;
    int q_col, k_col, v_col;
    const float* decay;         // [n][H*dim] decays
    float q_scale;
    float* state;               // [slots][H*vdim*dim]
    long long state_stride;
    const int* slots;
    const int* cu_seqlens;
    float* out;                 // [row slabs][n][H*vdim]
    long long out_slice;        // floats between the slices of two row slabs (set by gla_walk)
    int H, dim, vdim;
    int col_slabs;              // set by gla_walk
    // other uses of the walk: `qk_share` heads in a row read the same q and k (head h reads group h / qk_share; 1: every head
    // its own); `head_decay` [n][H] is one decay per token and head for all of a head's rows, `const_decay` [H] one per head
    // for all tokens (then `decay` is not read); `v_scale` [n][H] multiplies the head's v as it is read; the source has
    // `v_cols` columns per head, and columns v_cols .. vdim - 1 of S take a one (times v_scale) in v's place: their output is
    // the query's product with the decayed sum of the keys.  Null and v_cols = vdim: the ordinary forms.
    int qk_share;
    const float* head_decay;
    const float* const_decay;
    const float* v_scale;
    int v_cols;
};

// Launches the walk for n_seqs sequences of n_tokens tokens together; `rows` is what mlc_gla_rows gave; `silu`: q, k and v
// pass SiLU as they are read.  Returns 0 or an error code.
int gla_walk(GlaArgs a, int n_seqs, int n_tokens, int rows, bool silu, cudaStream_t s);

}  // namespace mlc
