// Two linear attentions whose memory decays per head, on the walk of linear_attention.cu:
//
// constant decay ("Lightning attention"): q, k, v pass SiLU;  S_t = decay_h S_{t-1} + k_t v_tᵀ,  o_t = S_tᵀ q_t.  Behind the
// walk the concatenated heads are divided by one root mean square, times a gain, times sigmoid of a gate.
//
// exponential gates (the matrix memory of xLSTM; Beck et al., "xLSTM: Extended Long Short-Term Memory"): per token and head a
// log input gate i = c · tanh(z_i / c) and a log forget gate f = logsigmoid(c · tanh(z_f / c)).  With a running maximum
//   m_t = max(f_t + m_{t-1}, i_t)        (m = 0 before the first token)
//   S_t = exp(f_t + m_{t-1} - m_t) S_{t-1} + exp(i_t - m_t) k_t v_tᵀ,   n_t the same with k_t alone,
//   o_t = S_tᵀ q_t / (max(|n_t · q_t|, exp(-m_t)) + 1e-6)
// n is one more column of S whose v is a one, so the walk carries it and n·q is that column's output.  m is a scan: a run of
// tokens acts on m as m -> max(A + m, B), and two such runs in a row are another; the scan's order of additions depends on
// the run's length, but whatever m it finds is used for the decay, the input's factor and the denominator alike, where it
// cancels.
//
// State, decays, gates and norms are float32 whatever the engine's type.
#include "common.cuh"
#include "linear_attention.cuh"

namespace mlc {

// ------------------------------------------------------------------ constant decay: what precedes the walk of a prompt
// SiLU on columns [0, width) of every row, in place.  (A step of few tokens leaves it to the walk, whose blocks then each do
// their own rows' and columns'; in a prompt every q and k would pass SiLU once per slab of columns.)
template <int VEC>
__global__ void silu_columns_kernel(float* __restrict__ rows, long long stride, int width, long long total) {
    const long long idx = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (idx >= total) return;
    const long long t = idx / width;
    float* p = rows + t * stride + (idx - t * width);
    if constexpr (VEC == 4) {
        float4 v = *reinterpret_cast<const float4*>(p);
        v.x = v.x / (1.0f + expf(-v.x)); v.y = v.y / (1.0f + expf(-v.y));
        v.z = v.z / (1.0f + expf(-v.z)); v.w = v.w / (1.0f + expf(-v.w));
        *reinterpret_cast<float4*>(p) = v;
    } else {
        p[0] = p[0] / (1.0f + expf(-p[0]));
    }
}

// ------------------------------------------------------------------ constant decay: what follows the walk
// out[t] = (sum of the walk's slices) / rms(row) · gain · sigmoid(gate) · out_scale.  A block per token, a thread PIECES
// pieces of VEC entries, the row in registers from its loads to its stores.
template <typename T, int VEC, int PIECES>
__global__ void __launch_bounds__(1024)
row_norm_gate_kernel(const float* __restrict__ o, int slices, long long slice_stride, const float* __restrict__ gate,
                     long long gate_stride, const float* __restrict__ gain, float eps, float out_scale, int inner,
                     T* __restrict__ out) {
    __shared__ float scratch[32];
    const long long t = blockIdx.x;
    const float* src = o + t * inner;
    const float* g = gate + t * gate_stride;
    float v[PIECES][VEC], z[PIECES][VEC], w[PIECES][VEC];
    float ss = 0.0f;
#pragma unroll
    for (int p = 0; p < PIECES; ++p) {
        const int c = (threadIdx.x + p * blockDim.x) * VEC;
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[p][k] = z[p][k] = w[p][k] = 0.0f;
        if (c >= inner) continue;
        if constexpr (VEC == 4) {
            const float4 a = *reinterpret_cast<const float4*>(g + c), b = *reinterpret_cast<const float4*>(gain + c);
            z[p][0] = a.x; z[p][1] = a.y; z[p][2] = a.z; z[p][3] = a.w;
            w[p][0] = b.x; w[p][1] = b.y; w[p][2] = b.z; w[p][3] = b.w;
            for (int s = 0; s < slices; ++s) {
                const float4 q = *reinterpret_cast<const float4*>(src + s * slice_stride + c);
                v[p][0] += q.x; v[p][1] += q.y; v[p][2] += q.z; v[p][3] += q.w;
            }
        } else {
            z[p][0] = g[c];
            w[p][0] = gain[c];
            for (int s = 0; s < slices; ++s) v[p][0] += src[s * slice_stride + c];
        }
#pragma unroll
        for (int k = 0; k < VEC; ++k) ss = fmaf(v[p][k], v[p][k], ss);
    }
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)inner + eps) * out_scale;
#pragma unroll
    for (int p = 0; p < PIECES; ++p) {
        const int c = (threadIdx.x + p * blockDim.x) * VEC;
        if (c >= inner) continue;
        float r[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) r[k] = v[p][k] * f * w[p][k] / (1.0f + expf(-z[p][k]));
        T* dst = out + t * inner + c;
        if constexpr (VEC == 4 && sizeof(T) == 4) {
            *reinterpret_cast<float4*>(dst) = make_float4(r[0], r[1], r[2], r[3]);
        } else if constexpr (VEC == 4) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
            *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
        } else {
            dst[0] = from_float<T>(r[0]);
        }
    }
}

// ------------------------------------------------------------------ exponential gates: decays and input factors
// zi, zf: the gates' logits with their biases
__device__ __forceinline__ void log_gates(float zi, float zf, float cap, float inv_cap, float& li, float& lf) {
    li = cap * tanhf(zi * inv_cap);
    const float x = cap * tanhf(zf * inv_cap);
    lf = fminf(x, 0.0f) - log1pf(expf(-fabsf(x)));
}

struct ExpGateArgs {
    const float* proj;          // rows with the gate logits at i_col + head and f_col + head
    long long stride;
    int i_col, f_col;
    const float* i_bias;        // [H]
    const float* f_bias;
    float cap, inv_cap;
    float* m_state;             // [slots][.]: H running maxima at the start of each slot's piece
    long long state_stride;
    const int* slots;
    const int* cu_seqlens;
    int H, n_seqs;
    float* decay;               // [n][H] exp(f + m_before - m)
    float* take;                // [n][H] exp(i - m)
    float* m_out;               // [n][H]
};

// Steps of one token per sequence: a thread per (sequence, head).
__global__ void exp_gates_step_kernel(ExpGateArgs a) {
    const int idx = blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= a.n_seqs * a.H) return;
    const int seq = idx / a.H, h = idx % a.H;
    float* ms = a.m_state + (long long)a.slots[seq] * a.state_stride + h;
    float m = *ms;
    for (int t = a.cu_seqlens[seq]; t < a.cu_seqlens[seq + 1]; ++t) {
        float li, lf;
        const float* row = a.proj + (long long)t * a.stride;
        log_gates(row[a.i_col + h] + a.i_bias[h], row[a.f_col + h] + a.f_bias[h], a.cap, a.inv_cap, li, lf);
        const float next = fmaxf(lf + m, li);
        const long long at = (long long)t * a.H + h;
        a.decay[at] = expf(lf + m - next);
        a.take[at] = expf(li - next);
        a.m_out[at] = next;
        m = next;
    }
    *ms = m;
}

// Longer runs: a block per (head, sequence) takes rounds of EG_THREADS x EG_RUN tokens, a thread EG_RUN tokens side by side.
constexpr int EG_THREADS = 512;
constexpr int EG_RUN = 4;

__global__ void __launch_bounds__(EG_THREADS)
exp_gates_scan_kernel(ExpGateArgs a) {
    __shared__ float wa[EG_THREADS / 32], wb[EG_THREADS / 32];
    __shared__ float carry;
    const int h = blockIdx.x, seq = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t0 = a.cu_seqlens[seq], t1 = a.cu_seqlens[seq + 1];
    float* ms = a.m_state + (long long)a.slots[seq] * a.state_stride + h;
    float m0 = *ms;
    const float bi = a.i_bias[h], bf = a.f_bias[h];
    for (int c0 = t0; c0 < t1; c0 += EG_THREADS * EG_RUN) {
        const int first = c0 + threadIdx.x * EG_RUN;
        float li[EG_RUN], lf[EG_RUN];
        float A = 0.0f, B = -INFINITY;                    // the thread's run: m -> max(A + m, B)
        float zi[EG_RUN], zf[EG_RUN];                     // all loads first (the last token's again where there is none)
#pragma unroll
        for (int u = 0; u < EG_RUN; ++u) {
            const float* row = a.proj + (long long)min(first + u, t1 - 1) * a.stride;
            zi[u] = row[a.i_col + h];
            zf[u] = row[a.f_col + h];
        }
#pragma unroll
        for (int u = 0; u < EG_RUN; ++u) {
            log_gates(zi[u] + bi, zf[u] + bf, a.cap, a.inv_cap, li[u], lf[u]);
            if (first + u >= t1) {
                li[u] = -INFINITY;
                lf[u] = 0.0f;                             // no token: m stays as it is
            }
        }
#pragma unroll
        for (int u = 0; u < EG_RUN; ++u) {
            A += lf[u];
            B = fmaxf(B + lf[u], li[u]);
        }
        // inclusive scan over the warp's threads, then over the warps' totals
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pa = __shfl_up_sync(0xffffffffu, A, o), pb = __shfl_up_sync(0xffffffffu, B, o);
            if (lane >= o) {
                B = fmaxf(pb + A, B);
                A += pa;
            }
        }
        if (lane == 31) {
            wa[warp] = A;
            wb[warp] = B;
        }
        float xa = __shfl_up_sync(0xffffffffu, A, 1), xb = __shfl_up_sync(0xffffffffu, B, 1);      // what lies before this thread in its warp
        if (lane == 0) {
            xa = 0.0f;
            xb = -INFINITY;
        }
        __syncthreads();
        float m = m0;
        for (int w = 0; w < warp; ++w) m = fmaxf(wa[w] + m, wb[w]);
        m = fmaxf(xa + m, xb);
#pragma unroll
        for (int u = 0; u < EG_RUN; ++u) {
            if (first + u >= t1) break;
            const float next = fmaxf(lf[u] + m, li[u]);
            const long long at = (long long)(first + u) * a.H + h;
            a.decay[at] = expf(lf[u] + m - next);
            a.take[at] = expf(li[u] - next);
            a.m_out[at] = next;
            m = next;
        }
        if (threadIdx.x == EG_THREADS - 1) carry = m;     // threads without tokens leave m as it is
        __syncthreads();
        m0 = carry;
    }
    if (threadIdx.x == 0 && t1 > t0) *ms = m0;
}

// Behind the walk: a warp per (token, head).  o holds vdim + 1 columns per head, the last one n·q.
//   y = o / (max(|n·q|, exp(-m)) + 1e-6);   out = y / rms(y) · gain · sigmoid(gate)
template <typename T, int PIECES>
__global__ void __launch_bounds__(128)
memory_finish_kernel(const float* __restrict__ o, int slices, long long slice_stride, const float* __restrict__ m,
                     const float* __restrict__ gate, long long gate_stride, const float* __restrict__ gain, float eps,
                     long long n_rows, int H, int vdim, T* __restrict__ out) {
    const long long row = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (row >= n_rows) return;
    const int lane = threadIdx.x & 31;
    const long long t = row / H;
    const int h = (int)(row - t * H);
    const float* src = o + row * (vdim + 1);
    const float* g = gate + t * gate_stride + (long long)h * vdim;
    const float* w = gain + (long long)h * vdim;
    float v[PIECES], z[PIECES], wv[PIECES];
#pragma unroll
    for (int k = 0; k < PIECES; ++k) {
        const int d = lane + 32 * k;
        v[k] = z[k] = wv[k] = 0.0f;
        if (d < vdim) {
            v[k] = src[d];
            z[k] = g[d];
            wv[k] = w[d];
        }
    }
    float nq = src[vdim];
    for (int s = 1; s < slices; ++s) {
        const float* p = src + s * slice_stride;
#pragma unroll
        for (int k = 0; k < PIECES; ++k)
            if (lane + 32 * k < vdim) v[k] += p[lane + 32 * k];
        nq += p[vdim];
    }
    const float size = 1.0f / (fmaxf(fabsf(nq), expf(-m[row])) + 1e-6f);
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < PIECES; ++k) {
        v[k] *= size;
        ss = fmaf(v[k], v[k], ss);
    }
    const float f = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
#pragma unroll
    for (int k = 0; k < PIECES; ++k) {
        const int d = lane + 32 * k;
        if (d < vdim) out[row * vdim + d] = from_float<T>(v[k] * f * wv[k] / (1.0f + expf(-z[k])));
    }
}

template <typename T>
static int launch_memory_finish(const float* o, int slices, long long slice_stride, const float* m, const float* gate,
                                long long gate_stride, const float* gain, float eps, long long n_rows, int H, int vdim, T* out,
                                cudaStream_t s) {
    const unsigned blocks = (unsigned)((n_rows + 3) / 4);
    auto k = vdim <= 64 ? memory_finish_kernel<T, 2> : vdim <= 128 ? memory_finish_kernel<T, 4> : vdim <= 256 ? memory_finish_kernel<T, 8>
           : vdim <= 512 ? memory_finish_kernel<T, 16> : memory_finish_kernel<T, 32>;
    k<<<blocks, 128, 0, s>>>(o, slices, slice_stride, m, gate, gate_stride, gain, eps, n_rows, H, vdim, out);
    MLC_LAUNCH_CHECK();
    return 0;
}

template <typename T>
static int launch_row_norm_gate(const float* o, int slices, long long slice_stride, const float* gate, long long gate_stride,
                                const float* gain, float eps, float out_scale, int n, int inner, T* out, cudaStream_t s) {
    const bool vec = (inner & 3) == 0 && (gate_stride & 3) == 0 &&
                     ((((uintptr_t)o) | ((uintptr_t)gate) | ((uintptr_t)gain) | ((uintptr_t)out)) & 15) == 0;
    const int items = vec ? inner / 4 : inner;
    int threads = (items + 31) / 32 * 32;
    if (threads > 1024) threads = 1024;
    const int pieces = (items + threads - 1) / threads;
    auto k = vec ? (pieces <= 1 ? row_norm_gate_kernel<T, 4, 1> : pieces <= 2 ? row_norm_gate_kernel<T, 4, 2> : row_norm_gate_kernel<T, 4, 4>)
                 : (pieces <= 2 ? row_norm_gate_kernel<T, 1, 2> : row_norm_gate_kernel<T, 1, 16>);
    k<<<n, threads, 0, s>>>(o, slices, slice_stride, gate, gate_stride, gain, eps, out_scale, inner, out);
    MLC_LAUNCH_CHECK();
    return 0;
}

}  // namespace mlc

using namespace mlc;

// Linear attention with a constant decay per head.  proj: float32 rows holding the logits of q, k (H x dim each) and v
// (H x vdim) side by side from column q_col on, and of the gate (H x vdim) at g_col; `silu_first` overwrites q, k and v with
// their SiLU (one more launch) instead of leaving it to the walk.  decay float32 [H], gain float32 [H*vdim].  state: float32, a slot's row holds
// H*vdim*dim floats ([head][column][row]).  rows: what mlc_gla_rows gave.  walk: float32 [ceil(dim / (8 * rows))][n][H*vdim]
// scratch.  out [n][H*vdim] of out_dtype.
extern "C" int mlc_decay_attention(float* proj, long long proj_stride, int q_col, int g_col, int silu_first,
                                   const float* decay, const float* gain, float eps, float out_scale, float* state,
                                   long long state_stride, const int* slots, const int* cu_seqlens, int n_seqs, int n_tokens,
                                   int H, int dim, int vdim, int rows, float* walk, void* out, int out_dtype, void* stream) {
    if (n_seqs <= 0 || n_tokens <= 0) return 0;
    if (H <= 0 || vdim <= 0 || (long long)H * vdim > 16384 || rows < 1) return MLC_ERR_BAD_SIZE;
    if (out_dtype != MLC_DTYPE_F32 && out_dtype != MLC_DTYPE_BF16) return MLC_ERR_BAD_DTYPE;
    cudaStream_t s = (cudaStream_t)stream;
    if (silu_first) {
        const int width = H * (2 * dim + vdim);
        const bool vec = (width & 3) == 0 && (proj_stride & 3) == 0 && (((uintptr_t)(proj + q_col)) & 15) == 0;
        const long long total = (long long)n_tokens * width, items = vec ? total / 4 : total;
        if (vec) silu_columns_kernel<4><<<(unsigned)((items + 255) / 256), 256, 0, s>>>(proj + q_col, proj_stride, width, total);
        else silu_columns_kernel<1><<<(unsigned)((items + 255) / 256), 256, 0, s>>>(proj + q_col, proj_stride, width, total);
        MLC_LAUNCH_CHECK();
    }
    GlaArgs a = {};
    a.qk = a.vsrc = proj; a.qk_stride = a.v_stride = proj_stride;
    a.q_col = q_col; a.k_col = q_col + H * dim; a.v_col = q_col + 2 * H * dim;
    a.const_decay = decay; a.q_scale = 1.0f;
    a.state = state; a.state_stride = state_stride; a.slots = slots; a.cu_seqlens = cu_seqlens; a.out = walk;
    a.H = H; a.dim = dim; a.vdim = a.v_cols = vdim; a.qk_share = 1;
    const int rc = gla_walk(a, n_seqs, n_tokens, rows, !silu_first, s);
    if (rc != 0) return rc;
    const int slices = (dim + 8 * rows - 1) / (8 * rows), inner = H * vdim;
    const long long slice = (long long)n_tokens * inner;
    return out_dtype == MLC_DTYPE_F32
               ? launch_row_norm_gate<float>(walk, slices, slice, proj + g_col, proj_stride, gain, eps, out_scale, n_tokens, inner, (float*)out, s)
               : launch_row_norm_gate<bf16>(walk, slices, slice, proj + g_col, proj_stride, gain, eps, out_scale, n_tokens, inner, (bf16*)out, s);
}

// The matrix memory with exponential gates.  proj: float32 rows holding q, k (H x dim each), v and the output gate (H x vdim
// each), the input and forget gates' logits (H each) at their columns.  i_bias, f_bias float32 [H], gain float32 [H*vdim].
// state: float32, a slot's row holds H*(vdim+1)*dim floats ([head][column][row], the last column n), then H running maxima.
// gates: float32 [3][n][H] scratch.  rows: what mlc_gla_rows gave for (n_seqs, H, dim, vdim + 1).  walk: float32
// [ceil(dim / (8 * rows))][n][H*(vdim+1)] scratch.  out [n][H*vdim] of out_dtype.  max_q_len: the longest run of a sequence.
extern "C" int mlc_matrix_memory(const float* proj, long long proj_stride, int q_col, int k_col, int v_col, int g_col, int i_col,
                                 int f_col, const float* i_bias, const float* f_bias, float cap, const float* gain, float eps,
                                 float* state, long long state_stride, const int* slots, const int* cu_seqlens, int n_seqs,
                                 int n_tokens, int max_q_len, int H, int dim, int vdim, int rows, float* gates, float* walk,
                                 void* out, int out_dtype, void* stream) {
    if (n_seqs <= 0 || n_tokens <= 0) return 0;
    if (H <= 0 || dim <= 0 || vdim <= 0 || vdim > 1024 || n_seqs > 65535 || rows < 1 || !(cap > 0.0f)) return MLC_ERR_BAD_SIZE;
    if (out_dtype != MLC_DTYPE_F32 && out_dtype != MLC_DTYPE_BF16) return MLC_ERR_BAD_DTYPE;
    cudaStream_t s = (cudaStream_t)stream;
    const long long per = (long long)n_tokens * H;
    float *decay = gates, *take = gates + per, *m = gates + 2 * per;
    const ExpGateArgs g{proj, proj_stride, i_col, f_col, i_bias, f_bias, cap, 1.0f / cap, state + (long long)H * (vdim + 1) * dim,
                        state_stride, slots, cu_seqlens, H, n_seqs, decay, take, m};
    if (max_q_len <= 4) exp_gates_step_kernel<<<(n_seqs * H + 63) / 64, 64, 0, s>>>(g);
    else exp_gates_scan_kernel<<<dim3(H, n_seqs), EG_THREADS, 0, s>>>(g);
    MLC_LAUNCH_CHECK();
    GlaArgs a = {};
    a.qk = a.vsrc = proj; a.qk_stride = a.v_stride = proj_stride;
    a.q_col = q_col; a.k_col = k_col; a.v_col = v_col;
    a.head_decay = decay; a.v_scale = take; a.q_scale = 1.0f / sqrtf((float)dim);
    a.state = state; a.state_stride = state_stride; a.slots = slots; a.cu_seqlens = cu_seqlens; a.out = walk;
    a.H = H; a.dim = dim; a.vdim = vdim + 1; a.v_cols = vdim; a.qk_share = 1;
    const int rc = gla_walk(a, n_seqs, n_tokens, rows, false, s);
    if (rc != 0) return rc;
    const int slices = (dim + 8 * rows - 1) / (8 * rows);
    const long long slice = per * (vdim + 1);
    return out_dtype == MLC_DTYPE_F32
               ? launch_memory_finish<float>(walk, slices, slice, m, proj + g_col, proj_stride, gain, eps, per, H, vdim, (float*)out, s)
               : launch_memory_finish<bf16>(walk, slices, slice, m, proj + g_col, proj_stride, gain, eps, per, H, vdim, (bf16*)out, s);
}
