// RMS norms that do more than one thing at once:
//
//   rms_pair      two norms of the same row: x (float32, the residual stream) takes what the layer before left (slices,
//                 a token's expert rows, or both), one root mean square is formed, and the row is written twice, each time
//                 with its own gain and in the engine's type: the inputs of two branches that both read x.
//   embed_rms     a row of the embedding table, normed as it is read, as the residual stream's first value.
//   diff_combine  what follows differential attention: the two maps' outputs of a head are subtracted, divided by the head's
//                 root mean square, scaled, and multiplied by the head's sigmoid gate.
//
// Statistics are float32: x / sqrt(mean(x²) + eps) · gain.
#include "common.cuh"
#include "norm_branch.cuh"

namespace mlc {

struct PairNorm {
    float* x;                   // [n][d]
    const float* gain1;
    const float* gain2;         // null: one norm only
    float eps;
    int d, n;
};

template <typename T, int VEC>
__device__ __forceinline__ void store_scaled(T* p, const float (&v)[VEC], float f, const float* gain) {
    if constexpr (VEC == 4) {
        const Four g = load_four(gain);
        const float r[4] = {v[0] * f * g.e[0], v[1] * f * g.e[1], v[2] * f * g.e[2], v[3] * f * g.e[3]};
        store_four<T>(p, r);
    } else {
        p[0] = from_float<T>(v[0] * f * gain[0]);
    }
}

// A block per row, the row in shared memory between the two passes.
template <typename T, int VEC>
__global__ void __launch_bounds__(1024)
rms_pair_kernel(PairNorm a, NormBranch br, T* __restrict__ out1, T* __restrict__ out2) {
    extern __shared__ __align__(16) float row[];
    __shared__ float scratch[32];
    grid_launch_dependents();
    grid_dependency_wait();
    const long long t = blockIdx.x, base = t * a.d;
    const bool has_branch = br.y != nullptr || br.rows != nullptr;
    float ss = 0.0f;
    for (int i = threadIdx.x * VEC; i < a.d; i += blockDim.x * VEC) {
        float v[VEC];
        if constexpr (VEC == 4) {
            const Four q = load_four(a.x + base + i);
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[k] = q.e[k];
        } else {
            v[0] = a.x[base + i];
        }
        if (has_branch) {
            add_branch<VEC>(br, t, a.d, i, v);
            if constexpr (VEC == 4) store_four<float>(a.x + base + i, v);
            else a.x[base + i] = v[0];
        }
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            row[i + k] = v[k];
            ss = fmaf(v[k], v[k], ss);
        }
    }
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)a.d + a.eps);
    for (int i = threadIdx.x * VEC; i < a.d; i += blockDim.x * VEC) {
        float v[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[k] = row[i + k];
        store_scaled<T, VEC>(out1 + base + i, v, f, a.gain1 + i);
        if (a.gain2 != nullptr) store_scaled<T, VEC>(out2 + base + i, v, f, a.gain2 + i);
    }
}

// Many rows: a warp per row, the row in registers (NV 16-byte pieces per lane, d <= 128 * NV, d a multiple of 4).
template <typename T, int NV>
__global__ void __launch_bounds__(256)
rms_pair_warp_kernel(PairNorm a, NormBranch br, T* __restrict__ out1, T* __restrict__ out2) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int lane = threadIdx.x & 31;
    const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (row >= a.n) return;
    const long long base = (long long)row * a.d;
    const int d4 = a.d >> 2;
    float4* x4 = reinterpret_cast<float4*>(a.x + base);
    float4 v[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        v[k] = i < d4 ? x4[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    if (br.y != nullptr) {
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
    if (br.rows != nullptr) {
        for (int j = 0; j < br.top; ++j) {
            const float w = br.weights[(long long)row * br.top + j];
            const float4* t4 = reinterpret_cast<const float4*>(br.rows + (long long)br.row_of[(long long)row * br.top + j] * a.d);
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
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < NV; ++k) ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    const float f = 1.0f / sqrtf(warp_sum(ss) / (float)a.d + a.eps);
    const bool has_branch = br.y != nullptr || br.rows != nullptr;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        if (i >= d4) continue;
        if (has_branch) x4[i] = v[k];
        const float r[4] = {v[k].x, v[k].y, v[k].z, v[k].w};
        store_scaled<T, 4>(out1 + base + 4 * i, r, f, a.gain1 + 4 * i);
        if (a.gain2 != nullptr) store_scaled<T, 4>(out2 + base + 4 * i, r, f, a.gain2 + 4 * i);
    }
}

static inline int row_block(int items) {
    int t = 32;
    while (t < items && t < 1024) t <<= 1;
    return t;
}

template <typename T>
static cudaError_t launch_rms_pair(const PairNorm& a, const NormBranch& br, T* out1, T* out2, cudaStream_t s) {
    const bool aligned = (a.d & 3) == 0 && ((((uintptr_t)a.x) | ((uintptr_t)br.y) | ((uintptr_t)br.rows) | ((uintptr_t)a.gain1) |
                                             ((uintptr_t)a.gain2) | ((uintptr_t)out1) | ((uintptr_t)out2)) & 15) == 0;
    const int nv = ((a.d >> 2) + 31) / 32;
    if (aligned && nv <= 12 && a.n >= 256) {
        auto k = nv <= 1 ? rms_pair_warp_kernel<T, 1> : nv <= 2 ? rms_pair_warp_kernel<T, 2> : nv <= 4 ? rms_pair_warp_kernel<T, 4>
               : nv <= 8 ? rms_pair_warp_kernel<T, 8> : rms_pair_warp_kernel<T, 12>;
        return launch_pdl(k, dim3((a.n + 7) / 8), dim3(256), 0, s, a, br, out1, out2);
    }
    const size_t smem = (size_t)a.d * sizeof(float);
    static bool raised = false;
    if (smem > 48 * 1024 && !raised) {
        for (auto k : {rms_pair_kernel<T, 1>, rms_pair_kernel<T, 4>}) {
            cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
            if (e != cudaSuccess) return e;
        }
        raised = true;
    }
    // few rows: one entry a thread has more loads in flight
    if (aligned && a.n >= 64) return launch_pdl(rms_pair_kernel<T, 4>, dim3(a.n), dim3(row_block(a.d >> 2)), smem, s, a, br, out1, out2);
    return launch_pdl(rms_pair_kernel<T, 1>, dim3(a.n), dim3(row_block(a.d)), smem, s, a, br, out1, out2);
}

// ------------------------------------------------------------------ embedding behind a norm
// A block per row, which it reads twice (the second time out of L1).
template <typename T>
__global__ void __launch_bounds__(1024)
embed_rms_kernel(const T* __restrict__ table, const int* __restrict__ ids, int d, float scale, const float* __restrict__ gain, float eps,
                 float* __restrict__ out) {
    __shared__ float scratch[32];
    grid_launch_dependents();
    grid_dependency_wait();
    const T* row = table + (long long)ids[blockIdx.x] * d;
    float* o = out + (long long)blockIdx.x * d;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        const float v = to_float(row[i]) * scale;
        ss = fmaf(v, v, ss);
    }
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += blockDim.x) o[i] = to_float(row[i]) * scale * f * gain[i];
}

// Many rows: a warp per row, the row in registers (NV pieces of four entries per lane, d <= 128 * NV, d a multiple of 4).
template <int NV>
__global__ void __launch_bounds__(256)
embed_rms_warp_kernel(const bf16* __restrict__ table, const int* __restrict__ ids, int n, int d, float scale,
                      const float* __restrict__ gain, float eps, float* __restrict__ out) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int lane = threadIdx.x & 31;
    const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (row >= n) return;
    const uint2* src = reinterpret_cast<const uint2*>(table + (long long)ids[row] * d);
    const int d4 = d >> 2;
    float v[NV][4];
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        const uint2 q = i < d4 ? src[i] : make_uint2(0u, 0u);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
        v[k][0] = a.x * scale; v[k][1] = a.y * scale; v[k][2] = b.x * scale; v[k][3] = b.y * scale;
        ss += (v[k][0] * v[k][0] + v[k][1] * v[k][1]) + (v[k][2] * v[k][2] + v[k][3] * v[k][3]);
    }
    const float f = 1.0f / sqrtf(warp_sum(ss) / (float)d + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        if (i >= d4) continue;
        store_scaled<float, 4>(out + (long long)row * d + 4 * i, v[k], f, gain + 4 * i);
    }
}

// ------------------------------------------------------------------ differential attention: what follows the two maps
// o: [n][H][2][D], a head's two outputs (vdim entries each, D >= vdim).  A warp per (token, head):
//   u = o1 - lambda · o2;   out = u / sqrt(mean(u²) + eps) · mult · sigmoid(gate[head])         (no gate: 1)
// VEC entries at a time, PIECES of them a lane.
template <typename T, int VEC>
__device__ __forceinline__ void load_pieces(const T* p, float (&v)[VEC]) {
    if constexpr (VEC == 1) {
        v[0] = to_float(p[0]);
    } else if constexpr (sizeof(T) == 4) {
        const Four q = load_four(reinterpret_cast<const float*>(p));
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[k] = q.e[k];
    } else {
        const uint2 q = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&q);
        const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
        v[0] = a.x; v[1 % VEC] = a.y; v[2 % VEC] = b.x; v[3 % VEC] = b.y;
    }
}

template <typename T, int VEC, int PIECES>
__global__ void __launch_bounds__(128)
diff_combine_kernel(const T* __restrict__ o, const float* __restrict__ gate, long long gate_stride, float lambda, float eps, float mult,
                    long long n_rows, int H, int vdim, int D, T* __restrict__ out) {
    const long long row = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (row >= n_rows) return;
    const int lane = threadIdx.x & 31;
    const T *p1 = o + row * 2 * D, *p2 = p1 + D;
    float u[PIECES][VEC];
    float ss = 0.0f;
    const float z = gate != nullptr ? gate[(row / H) * gate_stride + row % H] : 0.0f;
#pragma unroll
    for (int p = 0; p < PIECES; ++p) {
        const int c = (lane + 32 * p) * VEC;
#pragma unroll
        for (int k = 0; k < VEC; ++k) u[p][k] = 0.0f;
        if (c >= vdim) continue;
        float a[VEC], b[VEC];
        load_pieces<T, VEC>(p1 + c, a);
        load_pieces<T, VEC>(p2 + c, b);
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            u[p][k] = a[k] - lambda * b[k];
            ss = fmaf(u[p][k], u[p][k], ss);
        }
    }
    const float f = mult / sqrtf(warp_sum(ss) / (float)vdim + eps) * (gate != nullptr ? 1.0f / (1.0f + expf(-z)) : 1.0f);
#pragma unroll
    for (int p = 0; p < PIECES; ++p) {
        const int c = (lane + 32 * p) * VEC;
        if (c >= vdim) continue;
        T* dst = out + row * vdim + c;
        if constexpr (VEC == 4) {
            const float r[4] = {u[p][0] * f, u[p][1 % VEC] * f, u[p][2 % VEC] * f, u[p][3 % VEC] * f};
            store_four<T>(dst, r);
        } else {
            dst[0] = from_float<T>(u[p][0] * f);
        }
    }
}

template <typename T>
static int launch_diff_combine(const T* o, const float* gate, long long gate_stride, float lambda, float eps, float mult, long long n_rows,
                               int H, int vdim, int D, T* out, cudaStream_t s) {
    const bool vec = vdim >= 128 && (vdim & 3) == 0 && (D & 3) == 0 && ((((uintptr_t)o) | ((uintptr_t)out)) & 15) == 0;
    auto k = vec ? (vdim <= 128 ? diff_combine_kernel<T, 4, 1> : vdim <= 256 ? diff_combine_kernel<T, 4, 2> : diff_combine_kernel<T, 4, 4>)
                 : (vdim <= 64 ? diff_combine_kernel<T, 1, 2> : vdim <= 128 ? diff_combine_kernel<T, 1, 4> : diff_combine_kernel<T, 1, 16>);
    k<<<(unsigned)((n_rows + 3) / 4), 128, 0, s>>>(o, gate, gate_stride, lambda, eps, mult, n_rows, H, vdim, D, out);
    MLC_LAUNCH_CHECK();
    return 0;
}

}  // namespace mlc

using namespace mlc;

// x float32 [n][d] += y (n_slices slices of n·d floats, or null) + the tokens' expert rows (rows / row_of / weights / top, or
// null); out1 = x / rms(x) · gain1, and with gain2 out2 = x / rms(x) · gain2, both [n][d] of out_dtype.
extern "C" int mlc_rms_pair(float* x, const float* y, int n_slices, const float* rows, const int* row_of, const float* weights, int top,
                            const float* gain1, const float* gain2, float eps, int n, int d, void* out1, void* out2, int out_dtype,
                            void* stream) {
    if (n <= 0) return 0;
    if (d <= 0 || d > 32768 || (y != nullptr && n_slices < 1) || (rows != nullptr && (row_of == nullptr || weights == nullptr || top < 1)))
        return MLC_ERR_BAD_SIZE;
    if (gain1 == nullptr || out1 == nullptr || (gain2 == nullptr) != (out2 == nullptr)) return MLC_ERR_BAD_SIZE;
    const PairNorm a{x, gain1, gain2, eps, d, n};
    const NormBranch br{y, n_slices, (long long)n * d, rows, row_of, weights, top};
    cudaError_t e;
    if (out_dtype == MLC_DTYPE_F32) e = launch_rms_pair<float>(a, br, (float*)out1, (float*)out2, (cudaStream_t)stream);
    else if (out_dtype == MLC_DTYPE_BF16) e = launch_rms_pair<bf16>(a, br, (bf16*)out1, (bf16*)out2, (cudaStream_t)stream);
    else return MLC_ERR_BAD_DTYPE;
    return e == cudaSuccess ? 0 : (int)e;
}

// out[t] float32 = v / rms(v) · gain with v = table[ids[t]] · scale
extern "C" int mlc_embed_rms(const void* table, int table_dtype, const int* ids, int n, int d, float scale, const float* gain, float eps,
                             float* out, void* stream) {
    if (n <= 0) return 0;
    if (d <= 0) return MLC_ERR_BAD_SIZE;
    cudaError_t e;
    const int nv = ((d >> 2) + 31) / 32;
    if (table_dtype == MLC_DTYPE_BF16 && n >= 256 && (d & 3) == 0 && nv <= 32 &&
        ((((uintptr_t)table) | ((uintptr_t)gain) | ((uintptr_t)out)) & 15) == 0) {
        auto k = nv <= 4 ? embed_rms_warp_kernel<4> : nv <= 8 ? embed_rms_warp_kernel<8> : nv <= 16 ? embed_rms_warp_kernel<16> : embed_rms_warp_kernel<32>;
        e = launch_pdl(k, dim3((n + 7) / 8), dim3(256), 0, (cudaStream_t)stream, (const bf16*)table, ids, n, d, scale, gain, eps, out);
    } else if (table_dtype == MLC_DTYPE_F32)
        e = launch_pdl(embed_rms_kernel<float>, dim3(n), dim3(row_block(d)), 0, (cudaStream_t)stream, (const float*)table, ids, d, scale, gain, eps, out);
    else if (table_dtype == MLC_DTYPE_BF16)
        e = launch_pdl(embed_rms_kernel<bf16>, dim3(n), dim3(row_block(d)), 0, (cudaStream_t)stream, (const bf16*)table, ids, d, scale, gain, eps, out);
    else
        return MLC_ERR_BAD_DTYPE;
    return e == cudaSuccess ? 0 : (int)e;
}

// o [n][H][2][D] and out [n][H][vdim] of one type; gate: float32 rows with a logit per head (null: no gate)
extern "C" int mlc_diff_combine(const void* o, int dtype, const float* gate, long long gate_stride, float lambda, float eps, float mult,
                                int n, int H, int vdim, int D, void* out, void* stream) {
    if (n <= 0) return 0;
    if (H <= 0 || vdim <= 0 || D < vdim || vdim > 512) return MLC_ERR_BAD_SIZE;
    const long long rows = (long long)n * H;
    if (dtype == MLC_DTYPE_F32)
        return launch_diff_combine<float>((const float*)o, gate, gate_stride, lambda, eps, mult, rows, H, vdim, D, (float*)out, (cudaStream_t)stream);
    if (dtype == MLC_DTYPE_BF16)
        return launch_diff_combine<bf16>((const bf16*)o, gate, gate_stride, lambda, eps, mult, rows, H, vdim, D, (bf16*)out, (cudaStream_t)stream);
    return MLC_ERR_BAD_DTYPE;
}
