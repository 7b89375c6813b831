// A branch's output on its way into the residual stream, as the norm kernels read it: float32 slices added in order, or the
// weighted sum of a token's expert rows, sum_j weights[t][j] · rows[row_of[t][j]], j in the order of the choices.
#pragma once

#include "common.cuh"

namespace mlc {

struct NormBranch {
    const float* y;             // [n_slices][n][d], or null
    int n_slices;
    long long slice_stride;
    const float* rows;          // expert rows [.][d], or null
    const int* row_of;          // [n][top]
    const float* weights;       // [n][top]
    int top;
};

struct Four { float e[4]; };
__device__ __forceinline__ Four load_four(const float* p) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    return Four{{t.x, t.y, t.z, t.w}};
}

// v (VEC entries of row t from entry i on) += the branch's entries
template <int VEC>
__device__ __forceinline__ void add_branch(const NormBranch& br, long long t, int d, int i, float (&v)[VEC]) {
    if (br.y != nullptr) {
        const float* p = br.y + t * d + i;
#pragma unroll 8
        for (int s = 0; s < br.n_slices; ++s) {
            if constexpr (VEC == 4) {
                const Four q = load_four(p + s * br.slice_stride);
#pragma unroll
                for (int k = 0; k < VEC; ++k) v[k] += q.e[k];
            } else {
                v[0] += __ldg(p + s * br.slice_stride);
            }
        }
    }
    if (br.rows != nullptr) {
        float acc[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) acc[k] = 0.0f;
#pragma unroll 4
        for (int j = 0; j < br.top; ++j) {
            const float w = br.weights[t * br.top + j];
            const float* p = br.rows + (long long)br.row_of[t * br.top + j] * d + i;
            if constexpr (VEC == 4) {
                const Four q = load_four(p);
#pragma unroll
                for (int k = 0; k < VEC; ++k) acc[k] = fmaf(w, q.e[k], acc[k]);
            } else {
                acc[0] = fmaf(w, *p, acc[0]);
            }
        }
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[k] += acc[k];
    }
}

template <typename T>
__device__ __forceinline__ void store_four(T* p, const float (&r)[4]) {
    if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(r[0], r[1], r[2], r[3]);
    } else {
        __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
    }
}

}  // namespace mlc
