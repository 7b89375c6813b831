// Row-wise kernels around the matrix products: embedding gather, residual add fused with
// RMSNorm, the rotation table, the Q/K/V epilogue (bias, rotate-half RoPE, scatter of keys
// and values into the paged cache), SiLU(gate)·up, and row gather.
//
// The arithmetic follows the reference's scalar code and stays in float32 wherever the
// reference's does: the sum of squares and 1/sqrt(ss/d + eps) with the multiply order
// x·scale·w (src/ops.cpp:19-41), cos/sin of a float32 angle p·f_i and the pairing
// (i, i + hd/2) (src/ops.cpp:125-141), gate·(1/(1+exp(-gate)))·up (src/ops.cpp:94-107),
// the residual sum (src/forward.cpp:772, 779).  What is new is the fusion and the layout.
#include "common.cuh"
#include "norm_branch.cuh"

namespace mlc {

// ------------------------------------------------------------------ embedding
template <typename T>
__global__ void embed_kernel(const T* __restrict__ table, const int* __restrict__ ids, int d, float scale,
                             float* __restrict__ out) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int n = blockIdx.x;
    const T* row = table + (long long)ids[n] * d;
    float* o = out + (long long)n * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) o[i] = to_float(row[i]) * scale;
}

// ------------------------------------------------------------------ residual add + RMSNorm
// x (float32, the residual stream) += the sum of the delta slices, when given (a branch output,
// possibly left as split-K partial sums [n_slices][n][d]); out = x·scale·gain.
template <typename T>
__global__ void add_rmsnorm_kernel(float* __restrict__ x, const float* __restrict__ delta, int n_slices,
                                   long long slice_stride, const float* __restrict__ gain, float eps, int d,
                                   T* __restrict__ out) {
    __shared__ float scratch[32];
    grid_launch_dependents();
    grid_dependency_wait();
    const long long base = (long long)blockIdx.x * d;
    float ss = 0.0f;
    if (delta != nullptr) {
        for (int i = threadIdx.x; i < d; i += blockDim.x) {
            float v = x[base + i];
#pragma unroll 8
            for (int s = 0; s < n_slices; ++s) v += __ldg(delta + s * slice_stride + base + i);
            x[base + i] = v;
            ss += v * v;
        }
    } else {
        for (int i = threadIdx.x; i < d; i += blockDim.x) {
            const float v = x[base + i];
            ss += v * v;
        }
    }
    ss = block_sum(ss, scratch);
    const float scale = 1.0f / sqrtf(ss / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        out[base + i] = from_float<T>(x[base + i] * scale * gain[i]);
    }
}

// The same with 16-byte accesses, for rows whose length is a multiple of 4 (all pointers 16-byte aligned).
template <typename T>
__global__ void add_rmsnorm_vec4_kernel(float* __restrict__ x, const float* __restrict__ delta, int n_slices,
                                        long long slice_stride, const float* __restrict__ gain, float eps, int d,
                                        T* __restrict__ out) {
    __shared__ float scratch[32];
    grid_launch_dependents();
    grid_dependency_wait();
    const long long base = (long long)blockIdx.x * d;
    const int d4 = d >> 2;
    float4* x4 = reinterpret_cast<float4*>(x + base);
    float ss = 0.0f;
    for (int i = threadIdx.x; i < d4; i += blockDim.x) {
        float4 v = x4[i];
        if (delta != nullptr) {
#pragma unroll 4
            for (int s = 0; s < n_slices; ++s) {
                const float4 t = __ldg(reinterpret_cast<const float4*>(delta + s * slice_stride + base) + i);
                v.x += t.x; v.y += t.y; v.z += t.z; v.w += t.w;
            }
            x4[i] = v;
        }
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    ss = block_sum(ss, scratch);
    const float scale = 1.0f / sqrtf(ss / (float)d + eps);
    const float4* g4 = reinterpret_cast<const float4*>(gain);
    for (int i = threadIdx.x; i < d4; i += blockDim.x) {
        const float4 v = x4[i], g = __ldg(g4 + i);
        T* o = out + base + 4 * i;
        o[0] = from_float<T>(v.x * scale * g.x);
        o[1] = from_float<T>(v.y * scale * g.y);
        o[2] = from_float<T>(v.z * scale * g.z);
        o[3] = from_float<T>(v.w * scale * g.w);
    }
}

// Many rows (prompts): one warp per row, the row held in registers between the sum of squares and the scaling, so
// that every element is read once and the loads of a row are all in flight together; no block-wide barrier.
// NV = 16-byte pieces per lane (d <= 128 * NV).
template <typename T, int NV>
__global__ void __launch_bounds__(256)
add_rmsnorm_warp_kernel(float* __restrict__ x, const float* __restrict__ delta, int n_slices, long long slice_stride,
                        const float* __restrict__ gain, float eps, int d, int n, T* __restrict__ out) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int lane = threadIdx.x & 31;
    const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (row >= n) return;
    const long long base = (long long)row * d;
    const int d4 = d >> 2;
    float4* x4 = reinterpret_cast<float4*>(x + base);
    float4 v[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        v[k] = (i < d4) ? x4[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    if (delta != nullptr) {
        for (int s = 0; s < n_slices; ++s) {
            const float4* t4 = reinterpret_cast<const float4*>(delta + s * slice_stride + base);
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int i = lane + 32 * k;
                if (i < d4) {
                    const float4 t = __ldg(t4 + i);
                    v[k].x += t.x; v[k].y += t.y; v[k].z += t.z; v[k].w += t.w;
                }
            }
        }
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int i = lane + 32 * k;
            if (i < d4) x4[i] = v[k];
        }
    }
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < NV; ++k) ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    ss = warp_sum(ss);
    const float scale = 1.0f / sqrtf(ss / (float)d + eps);
    const float4* g4 = reinterpret_cast<const float4*>(gain);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        if (i < d4) {
            const float4 g = __ldg(g4 + i);
            const float a = v[k].x * scale * g.x, b = v[k].y * scale * g.y, c = v[k].z * scale * g.z, e = v[k].w * scale * g.w;
            if (sizeof(T) == 4) {
                reinterpret_cast<float4*>(out + base)[i] = make_float4(a, b, c, e);
            } else {
                __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, e);
                reinterpret_cast<uint2*>(out + base)[i] = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
            }
        }
    }
}

template <typename T>
static cudaError_t launch_rmsnorm_warp(int nv, float* x, const float* delta, int n_slices, long long stride, const float* gain,
                                       float eps, int d, int n, T* out, cudaStream_t s) {
    const dim3 grid((n + 7) / 8), block(256);
    switch (nv) {
        case 1: return launch_pdl(add_rmsnorm_warp_kernel<T, 1>, grid, block, 0, s, x, delta, n_slices, stride, gain, eps, d, n, out);
        case 2: return launch_pdl(add_rmsnorm_warp_kernel<T, 2>, grid, block, 0, s, x, delta, n_slices, stride, gain, eps, d, n, out);
        case 3: case 4: return launch_pdl(add_rmsnorm_warp_kernel<T, 4>, grid, block, 0, s, x, delta, n_slices, stride, gain, eps, d, n, out);
        case 5: case 6: case 7: case 8:
            return launch_pdl(add_rmsnorm_warp_kernel<T, 8>, grid, block, 0, s, x, delta, n_slices, stride, gain, eps, d, n, out);
        default: return launch_pdl(add_rmsnorm_warp_kernel<T, 16>, grid, block, 0, s, x, delta, n_slices, stride, gain, eps, d, n, out);
    }
}

// ------------------------------------------------------------------ rotation table
// table[p][i] = factor · (cos(p·f_i), sin(p·f_i)), the angle formed in float32 from an integer
// position and a float32 frequency, as src/ops.cpp:132-134 does for each token (factor 1 there;
// stretched rotations put a constant on both).
__global__ void rope_table_kernel(const float* __restrict__ inv_freq, int n_pos, int half, float factor,
                                  float2* __restrict__ table) {
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)n_pos * half) return;
    const int p = (int)(idx / half), i = (int)(idx % half);
    const float angle = (float)p * inv_freq[i];
    table[idx] = make_float2(cosf(angle) * factor, sinf(angle) * factor);
}

// ------------------------------------------------------------------ Q/K/V epilogue
// One block per token.  Input row: [q heads | k heads | v heads] in float32 straight from
// the projection.  Adds the bias, rotates q and k by the token's position, writes q as
// [token][head][hd] in the activation type and k, v into the token's place in the cache.
// With kv_heads_in_row == 0 the row holds q only (a layer that reads another's cache).
template <typename T>
__global__ void qkv_post_kernel(const float* __restrict__ qkv, const float* __restrict__ bias,
                                const int* __restrict__ positions, const int* __restrict__ tok_seq,
                                const float2* __restrict__ rope, int rope_positions, int q_heads,
                                int kv_heads_in_row, int hd, T* __restrict__ q_out, PagedKV cache) {
    const int n = blockIdx.x;
    const int half = hd >> 1;
    const int row_width = (q_heads + 2 * kv_heads_in_row) * hd;
    const float* row = qkv + (long long)n * row_width;
    const int p = positions[n];
    const int seq = tok_seq[n];
    const float2* cs = (rope != nullptr) ? rope + (long long)min(p, rope_positions - 1) * half : nullptr;

    // q and k heads: one thread per rotation pair
    const int rot_heads = q_heads + kv_heads_in_row;
    for (int idx = threadIdx.x; idx < rot_heads * half; idx += blockDim.x) {
        const int head = idx / half, i = idx % half;
        const int c0 = head * hd + i, c1 = c0 + half;
        float x0 = row[c0], x1 = row[c1];
        if (bias != nullptr) {
            x0 += bias[c0];
            x1 += bias[c1];
        }
        float y0 = x0, y1 = x1;
        if (cs != nullptr) {
            const float2 t = cs[i];
            y0 = x0 * t.x - x1 * t.y;
            y1 = x0 * t.y + x1 * t.x;
        }
        if (head < q_heads) {
            T* dst = q_out + ((long long)n * q_heads + head) * hd;
            dst[i] = from_float<T>(y0);
            dst[i + half] = from_float<T>(y1);
        } else {
            T* dst = (T*)cache.k_pool + paged_offset(cache, seq, p, head - q_heads);
            dst[i] = from_float<T>(y0);
            dst[i + half] = from_float<T>(y1);
        }
    }
    // v heads: bias only
    const int v_start = (q_heads + kv_heads_in_row) * hd;
    for (int idx = threadIdx.x; idx < kv_heads_in_row * hd; idx += blockDim.x) {
        const int head = idx / hd, i = idx % hd;
        float v = row[v_start + idx];
        if (bias != nullptr) v += bias[v_start + idx];
        T* dst = (T*)cache.v_pool + paged_offset(cache, seq, p, head);
        dst[i] = from_float<T>(v);
    }
}

// ------------------------------------------------------------------ SiLU(gate)·up
// Input row [gate (I) | up (I)], or with `interleaved` [g0, u0, g1, u1, ...]; output [I].
template <typename TIn, typename TOut>
__global__ void silu_mul_kernel(const TIn* __restrict__ gu, int inter, long long total, int interleaved,
                                TOut* __restrict__ out) {
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const long long n = idx / inter;
    const int i = (int)(idx % inter);
    const TIn* row = gu + n * 2 * inter;
    const float g = to_float(interleaved ? row[2 * i] : row[i]);
    const float u = to_float(interleaved ? row[2 * i + 1] : row[inter + i]);
    const float sig = 1.0f / (1.0f + expf(-g));
    out[idx] = from_float<TOut>(g * sig * u);
}

// Eight outputs per thread with 16-byte loads and stores (bfloat16 in and out, I a multiple of 8).
__global__ void silu_mul_vec8_kernel(const bf16* __restrict__ gu, int inter, long long total_vec, int interleaved,
                                     bf16* __restrict__ out) {
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total_vec) return;
    const int per_row = inter >> 3;
    const long long n = idx / per_row;
    const int i = (int)(idx % per_row) << 3;
    const bf16* row = gu + n * 2 * inter;
    float g[8], u[8];
    if (interleaved) {
        const uint4 a = *reinterpret_cast<const uint4*>(row + 2 * i);
        const uint4 b = *reinterpret_cast<const uint4*>(row + 2 * i + 8);
        const __nv_bfloat162* pa = reinterpret_cast<const __nv_bfloat162*>(&a);
        const __nv_bfloat162* pb = reinterpret_cast<const __nv_bfloat162*>(&b);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 fa = __bfloat1622float2(pa[k]), fb = __bfloat1622float2(pb[k]);
            g[k] = fa.x; u[k] = fa.y;
            g[4 + k] = fb.x; u[4 + k] = fb.y;
        }
    } else {
        const uint4 a = *reinterpret_cast<const uint4*>(row + i);
        const uint4 b = *reinterpret_cast<const uint4*>(row + inter + i);
        const __nv_bfloat162* pa = reinterpret_cast<const __nv_bfloat162*>(&a);
        const __nv_bfloat162* pb = reinterpret_cast<const __nv_bfloat162*>(&b);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 fa = __bfloat1622float2(pa[k]), fb = __bfloat1622float2(pb[k]);
            g[2 * k] = fa.x; g[2 * k + 1] = fa.y;
            u[2 * k] = fb.x; u[2 * k + 1] = fb.y;
        }
    }
    uint4 o;
    __nv_bfloat162* po = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const float y0 = g[2 * k] * (1.0f / (1.0f + expf(-g[2 * k]))) * u[2 * k];
        const float y1 = g[2 * k + 1] * (1.0f / (1.0f + expf(-g[2 * k + 1]))) * u[2 * k + 1];
        po[k] = __floats2bfloat162_rn(y0, y1);
    }
    *reinterpret_cast<uint4*>(out + n * inter + i) = o;
}

// ------------------------------------------------------------------ row gather
__global__ void gather_rows_kernel(const float* __restrict__ x, const float* __restrict__ delta, int n_slices,
                                   long long slice_stride, const int* __restrict__ rows, int d,
                                   float* __restrict__ out_x, float* __restrict__ out_delta) {
    grid_launch_dependents();
    grid_dependency_wait();
    const long long src = (long long)rows[blockIdx.x] * d, dst = (long long)blockIdx.x * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        out_x[dst + i] = x[src + i];
        if (delta != nullptr) {
            float v = 0.0f;
            for (int s = 0; s < n_slices; ++s) v += delta[s * slice_stride + src + i];
            out_delta[dst + i] = v;
        }
    }
}

// ------------------------------------------------------------------ dtype conversion
template <typename TIn, typename TOut>
__global__ void convert_kernel(const TIn* __restrict__ in, long long total, TOut* __restrict__ out) {
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx < total) out[idx] = from_float<TOut>(to_float(in[idx]));
}

// ------------------------------------------------------------------ layer norm (gain, optional bias)
// LN(v) = (v - mean(v)) / sqrt(mean((v - mean)²) + eps) · w + b, statistics in float32 in two passes (the mean first,
// then the squared deviations).  b may be null (no bias).
//
// ln_mode 0, "norm of the stream":   x += branch (if any);  out = LN(x)            (out in T)
// ln_mode 1, "norm of the branch":   x += LN(branch);       out = x, if asked for  (out in T)
//
// The branch: see norm_branch.cuh.
// A block per row; the row waits in shared memory between the passes.  VEC 4: 16-byte accesses (rows whose length is a
// multiple of 4, all pointers 16-byte aligned); VEC 1: any row, and few rows, where one entry a thread has more loads in flight.
template <typename T, int VEC>
__global__ void layernorm_kernel(float* __restrict__ x, NormBranch br, const float* __restrict__ gain,
                                 const float* __restrict__ bias, float eps, int d, int ln_mode, T* __restrict__ out) {
    extern __shared__ __align__(16) float row[];
    __shared__ float scratch[32];
    grid_launch_dependents();
    grid_dependency_wait();
    const long long t = blockIdx.x, base = t * d;
    const bool has_branch = br.y != nullptr || br.rows != nullptr;
    float sum = 0.0f;
    for (int i = threadIdx.x * VEC; i < d; i += blockDim.x * VEC) {
        float v[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[k] = 0.0f;
        if (ln_mode == 0) {
            if constexpr (VEC == 4) {
                const Four q = load_four(x + base + i);
#pragma unroll
                for (int k = 0; k < VEC; ++k) v[k] = q.e[k];
            } else {
                v[0] = x[base + i];
            }
        }
        if (has_branch) {
            add_branch<VEC>(br, t, d, i, v);
            if (ln_mode == 0) {
                if constexpr (VEC == 4) store_four<float>(x + base + i, v);
                else x[base + i] = v[0];
            }
        }
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            row[i + k] = v[k];
            sum += v[k];
        }
    }
    const float mean = block_sum(sum, scratch) / (float)d;
    float sq = 0.0f;
    for (int i = threadIdx.x * VEC; i < d; i += blockDim.x * VEC)
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            const float c = row[i + k] - mean;
            sq += c * c;
        }
    const float rstd = 1.0f / sqrtf(block_sum(sq, scratch) / (float)d + eps);
    for (int i = threadIdx.x * VEC; i < d; i += blockDim.x * VEC) {
        float r[VEC];
        if constexpr (VEC == 4) {
            const Four g = load_four(gain + i);
#pragma unroll
            for (int k = 0; k < VEC; ++k) r[k] = (row[i + k] - mean) * rstd * g.e[k];
            if (bias != nullptr) {
                const Four b = load_four(bias + i);
#pragma unroll
                for (int k = 0; k < VEC; ++k) r[k] += b.e[k];
            }
            if (ln_mode != 0) {
                const Four xo = load_four(x + base + i);
#pragma unroll
                for (int k = 0; k < VEC; ++k) r[k] = xo.e[k] + r[k];
                store_four<float>(x + base + i, r);
            }
            if (out != nullptr) store_four<T>(out + base + i, r);
        } else {
            r[0] = (row[i] - mean) * rstd * gain[i];
            if (bias != nullptr) r[0] += bias[i];
            if (ln_mode != 0) {
                r[0] = x[base + i] + r[0];
                x[base + i] = r[0];
            }
            if (out != nullptr) out[base + i] = from_float<T>(r[0]);
        }
    }
}

// Many rows: a warp per row, the row in registers from the first load to the last store (NV 16-byte pieces per lane,
// d <= 128 * NV, d a multiple of 4, all pointers 16-byte aligned).  The block's rows share gain and bias through shared
// memory, copied there asynchronously ahead of everything else (left to the last loop, their loads would wait one by one
// behind the row's registers).
// BRANCH: 0 none, 1 slices, 2 expert rows; MODE: ln_mode.  (Forms of their own: only what a form needs takes registers.)
template <typename T, int NV, int BRANCH, int MODE>
__global__ void __launch_bounds__(256)
layernorm_warp_kernel(float* __restrict__ x, NormBranch br, const float* __restrict__ gain, const float* __restrict__ bias,
                      float eps, int d, int n, T* __restrict__ out) {
    extern __shared__ __align__(16) float affine[];        // [d] gain, then [d] bias (if there is one)
    grid_launch_dependents();
    const int d4 = d >> 2;
    for (int i = threadIdx.x; i < (bias != nullptr ? 2 : 1) * d4; i += blockDim.x) {
        const float* src = i < d4 ? gain + 4 * i : bias + 4 * (i - d4);
        const unsigned dst = (unsigned)__cvta_generic_to_shared(affine + 4 * i);
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src));
    }
    asm volatile("cp.async.commit_group;\n" ::);
    grid_dependency_wait();
    const int lane = threadIdx.x & 31;
    const int row = min(blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), n - 1);
    const bool live = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5) < n;       // the last block's spare warps only keep company
    const long long base = (long long)row * d;
    float4* x4 = reinterpret_cast<float4*>(x + base);
    float4 v[NV], xv[MODE == 1 ? NV : 1];              // MODE 1 keeps the stream's entries beside the branch's
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        const float4 xi = live && i < d4 ? x4[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if constexpr (MODE == 0) {
            v[k] = xi;
        } else {
            xv[k] = xi;
            v[k] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
    }
    if constexpr (BRANCH == 1) {
        for (int s = 0; s < br.n_slices; ++s) {
            const float4* t4 = reinterpret_cast<const float4*>(br.y + s * br.slice_stride + base);
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int i = lane + 32 * k;
                if (i < d4) {
                    const float4 t = __ldg(t4 + i);
                    v[k].x += t.x; v[k].y += t.y; v[k].z += t.z; v[k].w += t.w;
                }
            }
        }
    }
    if constexpr (BRANCH == 2) {
        for (int j = 0; j < br.top; ++j) {
            const float w = br.weights[(long long)row * br.top + j];
            const float4* t4 = reinterpret_cast<const float4*>(br.rows + (long long)br.row_of[(long long)row * br.top + j] * d);
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int i = lane + 32 * k;
                if (i < d4) {
                    const float4 t = __ldg(t4 + i);
                    v[k].x = fmaf(w, t.x, v[k].x); v[k].y = fmaf(w, t.y, v[k].y);
                    v[k].z = fmaf(w, t.z, v[k].z); v[k].w = fmaf(w, t.w, v[k].w);
                }
            }
        }
    }
    float sum = 0.0f;
#pragma unroll
    for (int k = 0; k < NV; ++k) sum += (v[k].x + v[k].y) + (v[k].z + v[k].w);      // lanes beyond the row hold zeros
    const float mean = warp_sum(sum) / (float)d;
    float sq = 0.0f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        if (lane + 32 * k < d4) {
            const float a = v[k].x - mean, b = v[k].y - mean, c = v[k].z - mean, e = v[k].w - mean;
            sq += (a * a + b * b) + (c * c + e * e);
        }
    }
    const float rstd = 1.0f / sqrtf(warp_sum(sq) / (float)d + eps);
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();
    if (!live) return;
    const float4* g4 = reinterpret_cast<const float4*>(affine);
    const float4* b4 = bias != nullptr ? g4 + d4 : nullptr;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        if (i >= d4) continue;
        const float4 g = g4[i];
        float r[4] = {(v[k].x - mean) * rstd * g.x, (v[k].y - mean) * rstd * g.y, (v[k].z - mean) * rstd * g.z,
                      (v[k].w - mean) * rstd * g.w};
        if (b4 != nullptr) {
            const float4 b = b4[i];
            r[0] += b.x; r[1] += b.y; r[2] += b.z; r[3] += b.w;
        }
        if constexpr (MODE == 0) {
            if constexpr (BRANCH != 0) x4[i] = v[k];
        } else {
            r[0] += xv[k].x; r[1] += xv[k].y; r[2] += xv[k].z; r[3] += xv[k].w;
            x4[i] = make_float4(r[0], r[1], r[2], r[3]);
            if (out == nullptr) continue;
        }
        store_four<T>(out + base + 4 * i, r);
    }
}

template <typename T, int BRANCH, int MODE>
static cudaError_t launch_layernorm_warp(int nv, float* x, const NormBranch& br, const float* gain, const float* bias, float eps,
                                         int d, int n, T* out, cudaStream_t s) {
    auto k = nv <= 1 ? layernorm_warp_kernel<T, 1, BRANCH, MODE> : nv <= 2 ? layernorm_warp_kernel<T, 2, BRANCH, MODE>
           : nv <= 4 ? layernorm_warp_kernel<T, 4, BRANCH, MODE> : nv <= 8 ? layernorm_warp_kernel<T, 8, BRANCH, MODE>
           : layernorm_warp_kernel<T, 12, BRANCH, MODE>;
    return launch_pdl(k, dim3((n + 7) / 8), dim3(256), (size_t)d * sizeof(float) * (bias != nullptr ? 2 : 1), s, x, br,
                      gain, bias, eps, d, n, out);
}

template <typename T>
static cudaError_t launch_layernorm(bool vec, int nv, float* x, const NormBranch& br, const float* gain, const float* bias, float eps,
                                    int d, int n, int ln_mode, T* out, size_t smem, int threads, cudaStream_t s) {
    if (vec && nv <= 12 && n >= 128) {
        if (ln_mode == 0 && br.rows != nullptr) return launch_layernorm_warp<T, 2, 0>(nv, x, br, gain, bias, eps, d, n, out, s);
        if (ln_mode == 0 && br.y != nullptr) return launch_layernorm_warp<T, 1, 0>(nv, x, br, gain, bias, eps, d, n, out, s);
        if (ln_mode == 0) return launch_layernorm_warp<T, 0, 0>(nv, x, br, gain, bias, eps, d, n, out, s);
        if (br.rows != nullptr) return launch_layernorm_warp<T, 2, 1>(nv, x, br, gain, bias, eps, d, n, out, s);
        return launch_layernorm_warp<T, 1, 1>(nv, x, br, gain, bias, eps, d, n, out, s);
    }
    static bool raised = false;
    if (smem > 48 * 1024 && !raised) {
        for (auto k : {layernorm_kernel<T, 1>, layernorm_kernel<T, 4>}) {
            cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
            if (e != cudaSuccess) return e;
        }
        raised = true;
    }
    if (vec && n >= 128)
        return launch_pdl(layernorm_kernel<T, 4>, dim3(n), dim3(threads), smem, s, x, br, gain, bias, eps, d, ln_mode, out);
    return launch_pdl(layernorm_kernel<T, 1>, dim3(n), dim3(threads), smem, s, x, br, gain, bias, eps, d, ln_mode, out);
}

// ------------------------------------------------------------------ per-head RMS norm, partial rotation, cache write
// Rows of a projection in float32: q heads (H x dim) at q_col, k heads (KV x dim) at k_col, v heads (KV x vdim) at
// v_col.  q and k: each head divided by its root mean square over dim (eps inside the root) and multiplied by a gain
// shared by the heads (if given); then the first rot_dims entries of the head are rotated, entry i with entry
// i + rot_dims/2, by the token's row of the table ([positions][rot_dims/2] cos and sin, any factor on them already
// applied); the rest pass.  v is multiplied by v_scale.  q goes to q_out [token][head][D], k and v into the token's
// place in the cache, whose heads have D >= max(dim, vdim) entries: what lies beyond a head's own size is zero, which
// changes neither a score nor an output.  A warp per head.
// Options of the kernel below beyond its first form: biases added to the projection's columns as they are read (null:
// none); `whole_row`: the norm's statistic is taken over all query heads together (and over all key heads together) and the
// gains are as long as the projection, instead of one statistic per head and a gain shared by the heads; `interleaved`: the
// rotation pairs entry 2j with 2j + 1 instead of entry j with j + dims/2; `temp_every` > 0: the queries of position p are
// multiplied by 1 + temp_coef · ln(floor((p + 1) / temp_every) + 1).  `maps` > 1 (differential attention): a key head holds
// that many keys of `dim` entries side by side, each normed and rotated by itself, and query head h meets only the (h % maps)-th
// of them: its entries lie at that place of its row, zeros elsewhere.
struct QkOptions {
    const float* q_bias;
    const float* k_bias;
    const float* v_bias;
    int whole_row;
    int interleaved;
    float temp_coef;
    int temp_every;
    int maps;
};

template <typename T>
__global__ void qk_norm_rope_cache_kernel(const float* __restrict__ proj, long long stride, int q_col, int k_col, int v_col,
                                          const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps,
                                          const int* __restrict__ positions, const int* __restrict__ tok_seq,
                                          const float2* __restrict__ rope, int rope_positions, int rot_dims, int q_heads,
                                          int kv_heads_in_row, int dim, int vdim, int D, float v_scale, T* __restrict__ q_out,
                                          PagedKV cache, QkOptions opt) {
    const int n = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const float* row = proj + (long long)n * stride;
    const int p = positions[n];
    const int seq = tok_seq[n];
    const int half = rot_dims >> 1;
    const float2* cs = (rope != nullptr && half > 0) ? rope + (long long)min(p, rope_positions - 1) * half : nullptr;
    const int maps = opt.maps, k_units = maps * kv_heads_in_row;         // a unit: `dim` projected entries with a norm of their own
    const int n_heads = q_heads + k_units + kv_heads_in_row;
    const float q_temp = opt.temp_every > 0 ? 1.0f + opt.temp_coef * logf((float)((p + 1) / opt.temp_every) + 1.0f) : 1.0f;
    // a norm over the whole projection: one statistic for all query heads and one for all key heads, summed in an order
    // that the row's length alone fixes (a thread a strided share, then the block's tree)
    __shared__ float scratch[32];
    float f_q = 1.0f, f_k = 1.0f;
    if (opt.whole_row && eps >= 0.0f) {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < q_heads * dim; i += blockDim.x) {
            const float v = row[q_col + i] + (opt.q_bias != nullptr ? opt.q_bias[i] : 0.0f);
            ss += v * v;
        }
        f_q = 1.0f / sqrtf(block_sum(ss, scratch) / (float)(q_heads * dim) + eps);
        if (kv_heads_in_row > 0) {
            ss = 0.0f;
            for (int i = threadIdx.x; i < k_units * dim; i += blockDim.x) {
                const float v = row[k_col + i] + (opt.k_bias != nullptr ? opt.k_bias[i] : 0.0f);
                ss += v * v;
            }
            f_k = 1.0f / sqrtf(block_sum(ss, scratch) / (float)(k_units * dim) + eps);
        }
    }
    for (int head = warp; head < n_heads; head += n_warps) {
        if (head < q_heads + k_units) {
            const bool is_q = head < q_heads;
            const int h = is_q ? head : head - q_heads;
            const float* src = row + (is_q ? q_col : k_col) + h * dim;
            const float* bias = is_q ? opt.q_bias : opt.k_bias;
            if (bias != nullptr) bias += h * dim;
            const float* gain = is_q ? q_gain : k_gain;
            if (gain != nullptr && opt.whole_row) gain += h * dim;             // a gain as long as the projection
            T* dst = is_q ? q_out + ((long long)n * q_heads + head) * D
                          : (T*)cache.k_pool + paged_offset(cache, seq, p, h / maps);
            // the unit's place in its row, and the part of the row this unit writes (zeros where it has no entries)
            const int place = (h % maps) * dim;
            const int from = is_q ? 0 : place, to = is_q || h % maps == maps - 1 ? D : place + dim;
            float f = is_q ? f_q : f_k;
            if (!opt.whole_row) {
                float ss = 0.0f;
                for (int i = lane; i < dim; i += 32) {
                    const float v = src[i] + (bias != nullptr ? bias[i] : 0.0f);
                    ss += v * v;
                }
                ss = warp_sum(ss);
                f = eps >= 0.0f ? 1.0f / sqrtf(ss / (float)dim + eps) : 1.0f;      // a negative eps: no norm
            }
            if (is_q) f *= q_temp;              // the rotation is linear: the factor acts on both entries of a pair
            for (int at = from + lane; at < to; at += 32) {
                const int i = at - place;
                float v = 0.0f;
                if (i >= 0 && i < dim) {
                    const float raw = src[i] + (bias != nullptr ? bias[i] : 0.0f);
                    v = gain != nullptr ? raw * f * gain[i] : raw * f;
                    if (cs != nullptr && i < rot_dims) {
                        // the pair of entry i: i +- dims/2 (halves), or its neighbour 2j, 2j+1 (interleaved); the first of a
                        // pair becomes u cos - w sin, the second w cos + u sin
                        const bool first = opt.interleaved ? (i & 1) == 0 : i < half;
                        const int j = opt.interleaved ? i >> 1 : (i < half ? i : i - half);
                        const int partner = opt.interleaved ? (i ^ 1) : (i < half ? i + half : i - half);
                        const float praw = src[partner] + (bias != nullptr ? bias[partner] : 0.0f);
                        const float w = gain != nullptr ? praw * f * gain[partner] : praw * f;
                        const float2 t = cs[j];
                        v = first ? v * t.x - w * t.y : v * t.x + w * t.y;
                    }
                }
                dst[at] = from_float<T>(v);
            }
        } else {
            const int vh = head - q_heads - k_units;
            const float* src = row + v_col + vh * vdim;
            const float* bias = opt.v_bias != nullptr ? opt.v_bias + vh * vdim : nullptr;
            T* dst = (T*)cache.v_pool + paged_offset(cache, seq, p, vh);
            for (int i = lane; i < D; i += 32)
                dst[i] = from_float<T>(i < vdim ? (src[i] + (bias != nullptr ? bias[i] : 0.0f)) * v_scale : 0.0f);
        }
    }
}

// ------------------------------------------------------------------ soft cap: v <- c · tanh(v / c)
__global__ void softcap_kernel(float* __restrict__ v, long long total, float cap) {
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx < total) v[idx] = cap * tanhf(v[idx] / cap);
}

static inline int row_threads(int d) {
    int t = 32;
    while (t < d && t < 256) t <<= 1;
    return t;
}

// Few rows: one element per thread where the row allows it, so that every load of the row is in flight at once.
static inline int norm_threads(int d, int n) {
    if (n > 1024) return row_threads(d);
    int t = 32;
    while (t < d && t < 1024) t <<= 1;
    return t;
}

}  // namespace mlc

using namespace mlc;

// out[t] = table[ids[t]] · scale (a scale of one changes nothing, bit for bit)
extern "C" int mlc_embed(const void* table, int table_dtype, const int* ids, int n, int d, float scale, float* out,
                         void* stream) {
    if (n <= 0) return 0;
    if (d <= 0) return MLC_ERR_BAD_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    if (table_dtype == MLC_DTYPE_F32)
        e = launch_pdl(embed_kernel<float>, dim3(n), dim3(norm_threads(d, n)), 0, s, (const float*)table, ids, d, scale, out);
    else if (table_dtype == MLC_DTYPE_BF16)
        e = launch_pdl(embed_kernel<bf16>, dim3(n), dim3(norm_threads(d, n)), 0, s, (const bf16*)table, ids, d, scale, out);
    else
        return MLC_ERR_BAD_DTYPE;
    return e == cudaSuccess ? 0 : (int)e;
}

extern "C" int mlc_add_rmsnorm(float* x, const float* delta, int n_slices, const float* gain, float eps, int n, int d,
                               void* out, int out_dtype, void* stream) {
    if (n <= 0) return 0;
    if (d <= 0 || (delta != nullptr && n_slices < 1)) return MLC_ERR_BAD_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    const long long stride = (long long)n * d;
    cudaError_t e;
    const bool vec = (d & 3) == 0 && n > 64 &&
                     ((((uintptr_t)x) | ((uintptr_t)delta) | ((uintptr_t)gain) | ((uintptr_t)out)) & 15) == 0;
    const int nv = ((d >> 2) + 31) / 32;                 // 16-byte pieces per lane if a warp takes a row
    if (vec && nv <= 16 && n >= 256 && out_dtype == MLC_DTYPE_F32)
        e = launch_rmsnorm_warp<float>(nv, x, delta, n_slices, stride, gain, eps, d, n, (float*)out, s);
    else if (vec && nv <= 16 && n >= 256 && out_dtype == MLC_DTYPE_BF16)
        e = launch_rmsnorm_warp<bf16>(nv, x, delta, n_slices, stride, gain, eps, d, n, (bf16*)out, s);
    else if (vec && out_dtype == MLC_DTYPE_F32)
        e = launch_pdl(add_rmsnorm_vec4_kernel<float>, dim3(n), dim3(row_threads(d >> 2)), 0, s, x, delta, n_slices, stride, gain, eps, d, (float*)out);
    else if (vec && out_dtype == MLC_DTYPE_BF16)
        e = launch_pdl(add_rmsnorm_vec4_kernel<bf16>, dim3(n), dim3(row_threads(d >> 2)), 0, s, x, delta, n_slices, stride, gain, eps, d, (bf16*)out);
    else if (out_dtype == MLC_DTYPE_F32)
        e = launch_pdl(add_rmsnorm_kernel<float>, dim3(n), dim3(norm_threads(d, n)), 0, s, x, delta, n_slices, stride, gain, eps, d, (float*)out);
    else if (out_dtype == MLC_DTYPE_BF16)
        e = launch_pdl(add_rmsnorm_kernel<bf16>, dim3(n), dim3(norm_threads(d, n)), 0, s, x, delta, n_slices, stride, gain, eps, d, (bf16*)out);
    else
        return MLC_ERR_BAD_DTYPE;
    if (e != cudaSuccess) return (int)e;
    return 0;
}

// ln_mode 0: x += branch (if y or rows is given), out = LN(x)·gain + bias in out_dtype.
// ln_mode 1: x += LN(branch)·gain + bias; out (may be null) = the new x in out_dtype.
// The branch: y (n_slices slices of n·d floats), or rows / row_of / weights / top (a token's expert rows); bias may be null.
extern "C" int mlc_layernorm(float* x, const float* y, int n_slices, const float* rows, const int* row_of, const float* weights,
                             int top, const float* gain, const float* bias, float eps, int n, int d, int ln_mode, void* out,
                             int out_dtype, void* stream) {
    if (n <= 0) return 0;
    if (d <= 0 || d > 32768 || (y != nullptr && n_slices < 1) || (ln_mode != 0 && ln_mode != 1)) return MLC_ERR_BAD_SIZE;
    if (rows != nullptr && (y != nullptr || row_of == nullptr || weights == nullptr || top < 1)) return MLC_ERR_BAD_SIZE;
    if ((ln_mode == 1 && y == nullptr && rows == nullptr) || (ln_mode == 0 && out == nullptr)) return MLC_ERR_BAD_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    const NormBranch br{y, n_slices, (long long)n * d, rows, row_of, weights, top};
    const size_t smem = (size_t)d * sizeof(float);
    const int nv = ((d >> 2) + 31) / 32;                 // 16-byte pieces per lane if a warp takes a row
    const bool vec = (d & 3) == 0 && ((((uintptr_t)x) | ((uintptr_t)y) | ((uintptr_t)rows) | ((uintptr_t)gain) | ((uintptr_t)bias) |
                                       ((uintptr_t)out)) & 15) == 0;
    const int threads = vec && n >= 128 ? norm_threads(d >> 2, n) : norm_threads(d, n);
    cudaError_t e;
    if (out_dtype == MLC_DTYPE_F32)
        e = launch_layernorm<float>(vec, nv, x, br, gain, bias, eps, d, n, ln_mode, (float*)out, smem, threads, s);
    else if (out_dtype == MLC_DTYPE_BF16)
        e = launch_layernorm<bf16>(vec, nv, x, br, gain, bias, eps, d, n, ln_mode, (bf16*)out, smem, threads, s);
    else
        return MLC_ERR_BAD_DTYPE;
    return e == cudaSuccess ? 0 : (int)e;
}

extern "C" int mlc_qk_norm_rope_cache(const float* proj, long long stride, int q_col, int k_col, int v_col, const float* q_gain,
                                      const float* k_gain, float eps, const int* positions, const int* tok_seq,
                                      const void* rope_table, int rope_positions, int rot_dims, int n, int q_heads,
                                      int kv_heads_in_row, int dim, int vdim, int D, float v_scale, void* q_out, int dtype,
                                      void* k_pool, void* v_pool, const int* page_table, long long entry_offset,
                                      int pages_per_seq, int page_size, int cache_kv_heads, const float* q_bias,
                                      const float* k_bias, const float* v_bias, int whole_row, int interleaved, float temp_coef,
                                      int temp_every, int maps, void* stream) {
    if (n <= 0) return 0;
    const QkOptions opt{q_bias, k_bias, v_bias, whole_row, interleaved, temp_coef, temp_every, maps};
    if (maps < 1 || dim <= 0 || vdim <= 0 || D < maps * dim || D < vdim || q_heads <= 0 || q_heads % maps || kv_heads_in_row < 0) return MLC_ERR_BAD_SIZE;
    if (rot_dims < 0 || (rot_dims & 1) || rot_dims > dim) return MLC_ERR_BAD_SIZE;
    if (kv_heads_in_row != 0 && kv_heads_in_row != cache_kv_heads) return MLC_ERR_BAD_SIZE;
    PagedKV c{k_pool, v_pool, page_table, entry_offset, pages_per_seq, page_size, cache_kv_heads, D};
    cudaStream_t s = (cudaStream_t)stream;
    const int heads = q_heads + (maps + 1) * kv_heads_in_row;
    const int threads = 32 * (heads < 8 ? heads : 8);
    if (dtype == MLC_DTYPE_F32)
        qk_norm_rope_cache_kernel<float><<<n, threads, 0, s>>>(proj, stride, q_col, k_col, v_col, q_gain, k_gain, eps, positions,
                                                               tok_seq, (const float2*)rope_table, rope_positions, rot_dims, q_heads,
                                                               kv_heads_in_row, dim, vdim, D, v_scale, (float*)q_out, c, opt);
    else if (dtype == MLC_DTYPE_BF16)
        qk_norm_rope_cache_kernel<bf16><<<n, threads, 0, s>>>(proj, stride, q_col, k_col, v_col, q_gain, k_gain, eps, positions,
                                                              tok_seq, (const float2*)rope_table, rope_positions, rot_dims, q_heads,
                                                              kv_heads_in_row, dim, vdim, D, v_scale, (bf16*)q_out, c, opt);
    else
        return MLC_ERR_BAD_DTYPE;
    MLC_LAUNCH_CHECK();
    return 0;
}

extern "C" int mlc_softcap(float* v, long long total, float cap, void* stream) {
    if (total <= 0) return 0;
    if (!(cap > 0.0f)) return MLC_ERR_BAD_SIZE;
    softcap_kernel<<<(unsigned)((total + 255) / 256), 256, 0, (cudaStream_t)stream>>>(v, total, cap);
    MLC_LAUNCH_CHECK();
    return 0;
}

extern "C" int mlc_rope_table(const float* inv_freq, int n_pos, int half, float factor, void* table, void* stream) {
    if (n_pos <= 0 || half <= 0) return MLC_ERR_BAD_SIZE;
    const long long total = (long long)n_pos * half;
    rope_table_kernel<<<(unsigned)((total + 255) / 256), 256, 0, (cudaStream_t)stream>>>(inv_freq, n_pos, half, factor,
                                                                                         (float2*)table);
    MLC_LAUNCH_CHECK();
    return 0;
}

extern "C" int mlc_qkv_post(const float* qkv, const float* bias, const int* positions, const int* tok_seq,
                            const void* rope_table, int rope_positions, int n, int q_heads,
                            int kv_heads_in_row, int hd, void* q_out, int dtype, void* k_pool, void* v_pool,
                            const int* page_table, long long entry_offset, int pages_per_seq, int page_size,
                            int cache_kv_heads, void* stream) {
    if (n <= 0) return 0;
    if (hd <= 0 || (hd & 1) || q_heads <= 0 || kv_heads_in_row < 0) return MLC_ERR_BAD_SIZE;
    if (kv_heads_in_row != 0 && kv_heads_in_row != cache_kv_heads) return MLC_ERR_BAD_SIZE;
    PagedKV c{k_pool, v_pool, page_table, entry_offset, pages_per_seq, page_size, cache_kv_heads, hd};
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = row_threads((q_heads + kv_heads_in_row) * hd / 2);
    if (dtype == MLC_DTYPE_F32)
        qkv_post_kernel<float><<<n, threads, 0, s>>>(qkv, bias, positions, tok_seq, (const float2*)rope_table,
                                                     rope_positions, q_heads, kv_heads_in_row, hd,
                                                     (float*)q_out, c);
    else if (dtype == MLC_DTYPE_BF16)
        qkv_post_kernel<bf16><<<n, threads, 0, s>>>(qkv, bias, positions, tok_seq, (const float2*)rope_table,
                                                    rope_positions, q_heads, kv_heads_in_row, hd, (bf16*)q_out,
                                                    c);
    else
        return MLC_ERR_BAD_DTYPE;
    MLC_LAUNCH_CHECK();
    return 0;
}

extern "C" int mlc_silu_mul(const void* gate_up, int in_dtype, int n, int inter, int interleaved, void* out,
                            int out_dtype, void* stream) {
    if (n <= 0) return 0;
    if (inter <= 0) return MLC_ERR_BAD_SIZE;
    const long long total = (long long)n * inter;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    cudaStream_t s = (cudaStream_t)stream;
    if (in_dtype == MLC_DTYPE_BF16 && out_dtype == MLC_DTYPE_BF16 && (inter & 7) == 0 &&
        ((((uintptr_t)gate_up) | ((uintptr_t)out)) & 15) == 0) {
        const long long total_vec = total >> 3;
        silu_mul_vec8_kernel<<<(unsigned)((total_vec + 255) / 256), 256, 0, s>>>((const bf16*)gate_up, inter, total_vec,
                                                                                 interleaved, (bf16*)out);
        MLC_LAUNCH_CHECK();
        return 0;
    }
    if (in_dtype == MLC_DTYPE_F32 && out_dtype == MLC_DTYPE_F32)
        silu_mul_kernel<float, float><<<blocks, 256, 0, s>>>((const float*)gate_up, inter, total, interleaved, (float*)out);
    else if (in_dtype == MLC_DTYPE_F32 && out_dtype == MLC_DTYPE_BF16)
        silu_mul_kernel<float, bf16><<<blocks, 256, 0, s>>>((const float*)gate_up, inter, total, interleaved, (bf16*)out);
    else if (in_dtype == MLC_DTYPE_BF16 && out_dtype == MLC_DTYPE_BF16)
        silu_mul_kernel<bf16, bf16><<<blocks, 256, 0, s>>>((const bf16*)gate_up, inter, total, interleaved, (bf16*)out);
    else if (in_dtype == MLC_DTYPE_BF16 && out_dtype == MLC_DTYPE_F32)
        silu_mul_kernel<bf16, float><<<blocks, 256, 0, s>>>((const bf16*)gate_up, inter, total, interleaved, (float*)out);
    else
        return MLC_ERR_BAD_DTYPE;
    MLC_LAUNCH_CHECK();
    return 0;
}

extern "C" int mlc_gather_rows(const float* x, const float* delta, int n_slices, long long slice_stride, const int* rows,
                               int n_rows, int d, float* out_x, float* out_delta, void* stream) {
    if (n_rows <= 0) return 0;
    cudaError_t e = launch_pdl(gather_rows_kernel, dim3(n_rows), dim3(norm_threads(d, n_rows)), 0, (cudaStream_t)stream, x, delta,
                               n_slices, slice_stride, rows, d, out_x, out_delta);
    return e == cudaSuccess ? 0 : (int)e;
}

extern "C" int mlc_convert(const void* in, int in_dtype, long long total, void* out, int out_dtype, void* stream) {
    if (total <= 0) return 0;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    cudaStream_t s = (cudaStream_t)stream;
    if (in_dtype == MLC_DTYPE_F32 && out_dtype == MLC_DTYPE_BF16)
        convert_kernel<float, bf16><<<blocks, 256, 0, s>>>((const float*)in, total, (bf16*)out);
    else if (in_dtype == MLC_DTYPE_BF16 && out_dtype == MLC_DTYPE_F32)
        convert_kernel<bf16, float><<<blocks, 256, 0, s>>>((const bf16*)in, total, (float*)out);
    else
        return MLC_ERR_BAD_DTYPE;
    MLC_LAUNCH_CHECK();
    return 0;
}

// Switch programmatic dependent launch on (1, the default) or off (0) for this library's kernels.
extern "C" int mlc_set_pdl(int enabled) {
    mlc::pdl_enabled() = enabled ? 1 : 0;
    return 0;
}

// A copy between pinned host memory and the device on the given stream, for the few hundred bytes a decode step
// brings and takes: the call costs the host a third of what a tensor library's copy does.  direction 0: host to
// device, 1: device to host.
extern "C" int mlc_copy_async(void* dst, const void* src, long long bytes, int direction, void* stream) {
    if (bytes <= 0) return 0;
    if (dst == nullptr || src == nullptr || (direction != 0 && direction != 1)) return MLC_ERR_BAD_SIZE;
    cudaError_t e = cudaMemcpyAsync(dst, src, (size_t)bytes, direction == 0 ? cudaMemcpyHostToDevice : cudaMemcpyDeviceToHost,
                                    (cudaStream_t)stream);
    return e == cudaSuccess ? 0 : (int)e;
}
