// Latent attention: keys and values of all heads are expansions of one normed low-rank latent c per token, beside one
// rotated key part that the heads share.  Only [c | rotated part] is cached, one row per token, and attention runs
// on the cached rows themselves:
//
//   score_h(i, j) = (W_uk,hᵀ q_plain,h(i)) · c(j) + q_rot,h(i) · k_rot(j)         the key expansion moved to the query
//   out_h(i)      = W_uv,h (sum_j p_h(i, j) c(j))                                  the value expansion moved behind the sum
//
// which is attention with one key/value head of size rank + rot that every query head reads, values being the first
// `rank` entries of the key rows.  Two kernels here: `latent_prepare` (norm of the latent, rotation of the shared key
// part and of the queries' rotated parts, the cache write) and `head_project` (a small matrix product per head, for
// the two moved expansions), both with float32 arithmetic.  `head_project` has a second form for 16-bit weights on the
// tensor cores (mma.sync: the operands are a few megabytes at most, so what counts is that every load of a tile is in flight
// at once); its float32 inputs enter as the sum of two 16-bit numbers.
#include "common.cuh"

namespace mlc {

// A block per token.  proj row: q heads ([dim plain | rot rotated] each) at q_col, then [rank latent | rot] at kv_col.
// Cache row (kv head 0): [c · (rsqrt(mean c² + eps) · gain) | rotated key part | zeros up to D].
// q_out [n][H][D]: entries [rank, rank + rot) get the rotated query part, [rank + rot, D) zeros; [0, rank) is left to
// the projection that follows.  q_plain_out [n][H][dim] float32: the unrotated query parts, dense.
// `qsrc` (row stride `q_stride`) holds the query heads at q_col; it may be `proj` itself or another matrix (queries that
// come out of a product of their own, behind a query latent).  `interleaved`: the rotation pairs entry 2i with 2i + 1
// instead of i with i + rot/2; the table is the same, [position][pair] (cos, sin).
template <typename T>
__global__ void latent_prepare_kernel(const float* __restrict__ proj, long long stride, const float* __restrict__ qsrc,
                                      long long q_stride, int interleaved, int q_col, int kv_col,
                                      const float* __restrict__ gain, float eps, const int* __restrict__ positions,
                                      const int* __restrict__ tok_seq, const float2* __restrict__ rope, int rope_positions,
                                      int H, int dim, int rot, int rank, int D, T* __restrict__ q_out, int write_cache,
                                      PagedKV cache) {
    const int n = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const float* row = proj + (long long)n * stride;
    const int p = positions[n];
    const int half = rot >> 1;
    const float2* cs = (rope != nullptr && half > 0) ? rope + (long long)min(p, rope_positions - 1) * half : nullptr;
    for (int head = warp; head < H + 1; head += n_warps) {
        if (head < H) {
            const float* src = qsrc + (long long)n * q_stride + q_col + (long long)head * (dim + rot) + dim;
            T* dst = q_out + ((long long)n * H + head) * D + rank;
            for (int i = lane; i < D - rank; i += 32) {
                float v = 0.0f;
                if (i < rot) {
                    v = src[i];
                    if (cs != nullptr) {
                        const bool first = interleaved ? !(i & 1) : i < half;
                        const int j = interleaved ? i >> 1 : (i < half ? i : i - half);
                        const float w = src[interleaved ? i ^ 1 : (i < half ? i + half : i - half)];
                        const float2 t = cs[j];
                        v = first ? v * t.x - w * t.y : v * t.x + w * t.y;
                    }
                }
                dst[i] = from_float<T>(v);
            }
        } else if (write_cache) {
            const float* src = row + kv_col;
            T* dst = (T*)cache.k_pool + paged_offset(cache, tok_seq[n], p, 0);
            float ss = 0.0f;
            for (int i = lane; i < rank; i += 32) ss += src[i] * src[i];
            ss = warp_sum(ss);
            const float f = 1.0f / sqrtf(ss / (float)rank + eps);
            for (int i = lane; i < D; i += 32) {
                float v = 0.0f;
                if (i < rank) {
                    v = src[i] * f * gain[i];
                } else if (i < rank + rot) {
                    const int k = i - rank;
                    v = src[i];
                    if (cs != nullptr) {
                        const bool first = interleaved ? !(k & 1) : k < half;
                        const int j = interleaved ? k >> 1 : (k < half ? k : k - half);
                        const float w = src[rank + (interleaved ? k ^ 1 : (k < half ? k + half : k - half))];
                        const float2 t = cs[j];
                        v = first ? v * t.x - w * t.y : v * t.x + w * t.y;
                    }
                }
                dst[i] = from_float<T>(v);
            }
        }
    }
}

constexpr int HP_TILE = 64;
constexpr int HP_K = 16;

// out[t][h][j] = sum_d in[t][h][d] · W[h][d][j] for j < n_out, d < n_in; every operand by strides (in elements):
// in at t*in_st + h*in_sh + d, W at h*w_sh + d*w_sd + j*w_sj, out at t*out_st + h*out_sh + j.
// `gate` (float32 rows of stride gate_st, or null): out is multiplied by sigmoid(gate[t][h*n_out + j]) before it is rounded.
template <typename TI, typename TW, typename TO>
__global__ void __launch_bounds__(256)
head_project_kernel(const TI* __restrict__ in, long long in_st, long long in_sh, const TW* __restrict__ w, long long w_sh,
                    long long w_sd, long long w_sj, TO* __restrict__ out, long long out_st, long long out_sh, int n, int n_in,
                    int n_out, const float* __restrict__ gate, long long gate_st) {
    const int h = blockIdx.z;
    const int t0 = blockIdx.y * HP_TILE, j0 = blockIdx.x * HP_TILE;
    __shared__ float xs[HP_K][HP_TILE + 1];
    __shared__ float ws[HP_K][HP_TILE + 1];
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;
    for (int d0 = 0; d0 < n_in; d0 += HP_K) {
        for (int idx = threadIdx.x; idx < HP_TILE * HP_K; idx += 256) {
            const int r = idx / HP_K, k = idx % HP_K;
            xs[k][r] = (t0 + r < n && d0 + k < n_in) ? to_float(in[(long long)(t0 + r) * in_st + h * in_sh + d0 + k]) : 0.0f;
            // W: walk it the way it lies in memory
            const int rr = w_sj == 1 ? idx % HP_TILE : r, kk = w_sj == 1 ? idx / HP_TILE : k;
            ws[kk][rr] = (j0 + rr < n_out && d0 + kk < n_in) ? to_float(w[h * w_sh + (long long)(d0 + kk) * w_sd + (long long)(j0 + rr) * w_sj]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < HP_K; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = xs[k][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = ws[k][tx * 4 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= n) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = j0 + tx * 4 + j;
            if (c >= n_out) continue;
            float v = acc[i][j];
            if (gate != nullptr) v /= 1.0f + expf(-gate[t * gate_st + (long long)h * n_out + c]);
            out[(long long)t * out_st + h * out_sh + c] = from_float<TO>(v);
        }
    }
}

// ---- the same product on the tensor cores: W in bfloat16, accumulation in float32.
__device__ __forceinline__ void hp_ldmatrix(unsigned (&r)[4], const bf16* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void hp_ldmatrix_trans(unsigned (&r)[4], const bf16* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void hp_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct HeadProjectArgs {
    const void* in;
    long long in_st, in_sh;
    const bf16* w;
    long long w_sh;
    long long w_ld;             // elements between W's rows: [j][d] rows of d, or [d][j] rows of j
    bf16* out;
    long long out_st, out_sh;
    int n, n_in, n_out;
    const float* gate;
    long long gate_st;
};

// A block: TM tokens x 64 outputs of one head, four warps.  TM = 64: warp w takes tokens 16w .. 16w+15 and all 64 outputs;
// TM = 16: all warps take the 16 tokens, warp w outputs 16w .. 16w+15.  The inner size is walked in chunks of KC, each staged
// in shared memory by 16-byte loads (sizes, strides and addresses allow them: the host sees to it).  A float32 input x is
// staged as hi + lo, hi = x rounded to bfloat16 and lo = x - hi rounded, and both meet the weights.  An output's products are
// added in the same order whatever TM.  BY_D: W's rows hold d contiguously ([j][d]); else [d][j].
template <typename TI, int TM, bool BY_D>
__global__ void __launch_bounds__(128)
head_project_mma_kernel(HeadProjectArgs a) {
    constexpr int KC = TM == 16 ? 128 : 64;
    constexpr int XS = KC + 8, WS = BY_D ? KC + 8 : 64 + 8;
    constexpr bool SPLIT = sizeof(TI) == 4;
    constexpr int NT = TM == 16 ? 1 : 4;                   // pairs of 8-output tiles a warp owns
    __shared__ __align__(16) bf16 xs[(SPLIT ? 2 : 1) * TM * XS];
    __shared__ __align__(16) bf16 ws[BY_D ? 64 * WS : KC * WS];
    const int h = blockIdx.z, t0 = blockIdx.y * TM, j0 = blockIdx.x * 64;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int row0 = TM == 16 ? 0 : 16 * warp, col0 = TM == 16 ? 16 * warp : 0;
    const TI* in = (const TI*)a.in + (long long)h * a.in_sh;
    const bf16* w = a.w + (long long)h * a.w_sh;
    float acc[2 * NT][4];
#pragma unroll
    for (int i = 0; i < 2 * NT; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) acc[i][k] = 0.0f;
    grid_launch_dependents();
    for (int d0 = 0; d0 < a.n_in; d0 += KC) {
        if (d0 > 0) __syncthreads();
        // the weights' chunk: they depend on no kernel before this one
        constexpr int W_ROWS = BY_D ? 64 : KC, W_PACKS = (BY_D ? KC : 64) / 8;
#pragma unroll
        for (int idx = tid; idx < W_ROWS * W_PACKS; idx += 128) {
            const int r = idx / W_PACKS, c = (idx % W_PACKS) * 8;
            const int j = j0 + (BY_D ? r : c), d = d0 + (BY_D ? c : r);
            uint4 v = make_uint4(0, 0, 0, 0);
            if (j < a.n_out && d < a.n_in) v = *reinterpret_cast<const uint4*>(w + (BY_D ? j * a.w_ld + d : d * a.w_ld + j));
            *reinterpret_cast<uint4*>(ws + r * WS + c) = v;
        }
        if (d0 == 0) grid_dependency_wait();
#pragma unroll
        for (int idx = tid; idx < TM * (KC / 8); idx += 128) {
            const int r = idx / (KC / 8), c = (idx % (KC / 8)) * 8;
            const bool ok = t0 + r < a.n && d0 + c < a.n_in;
            const TI* p = in + (long long)(t0 + r) * a.in_st + d0 + c;
            if constexpr (SPLIT) {
                float4 u = make_float4(0.0f, 0.0f, 0.0f, 0.0f), v = u;
                if (ok) {
                    u = *reinterpret_cast<const float4*>(p);
                    v = *reinterpret_cast<const float4*>(p + 4);
                }
                const float f[8] = {u.x, u.y, u.z, u.w, v.x, v.y, v.z, v.w};
                __align__(16) bf16 hi[8], lo[8];
#pragma unroll
                for (int k = 0; k < 8; ++k) {
                    hi[k] = __float2bfloat16_rn(f[k]);
                    lo[k] = __float2bfloat16_rn(f[k] - __bfloat162float(hi[k]));
                }
                *reinterpret_cast<uint4*>(xs + r * XS + c) = *reinterpret_cast<const uint4*>(hi);
                *reinterpret_cast<uint4*>(xs + (TM + r) * XS + c) = *reinterpret_cast<const uint4*>(lo);
            } else {
                uint4 v = make_uint4(0, 0, 0, 0);
                if (ok) v = *reinterpret_cast<const uint4*>(p);
                *reinterpret_cast<uint4*>(xs + r * XS + c) = v;
            }
        }
        __syncthreads();
        const int k_end = min(KC, (a.n_in - d0 + 15) & ~15);       // what lies beyond n_in is zero
        for (int k = 0; k < k_end; k += 16) {
            unsigned ah[4], al[4];
            hp_ldmatrix(ah, xs + (row0 + (lane & 15)) * XS + k + (lane >> 4) * 8);
            if constexpr (SPLIT) hp_ldmatrix(al, xs + (TM + row0 + (lane & 15)) * XS + k + (lane >> 4) * 8);
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                unsigned b[4];
                const int c = col0 + 16 * t;
                if constexpr (BY_D) hp_ldmatrix(b, ws + (c + (lane >> 4) * 8 + (lane & 7)) * WS + k + ((lane >> 3) & 1) * 8);
                else hp_ldmatrix_trans(b, ws + (k + (lane & 15)) * WS + c + (lane >> 4) * 8);
                hp_mma(acc[2 * t], ah, b[0], b[1]);
                hp_mma(acc[2 * t + 1], ah, b[2], b[3]);
                if constexpr (SPLIT) {
                    hp_mma(acc[2 * t], al, b[0], b[1]);
                    hp_mma(acc[2 * t + 1], al, b[2], b[3]);
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 2 * NT; ++i) {
        const int j = j0 + col0 + 8 * i + (lane & 3) * 2;
        if (j >= a.n_out) continue;                        // n_out is even
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int t = t0 + row0 + (lane >> 2) + 8 * half;
            if (t >= a.n) continue;
            float u = acc[i][2 * half], v = acc[i][2 * half + 1];
            if (a.gate != nullptr) {
                const float* g = a.gate + t * a.gate_st + (long long)h * a.n_out + j;
                u /= 1.0f + expf(-g[0]);
                v /= 1.0f + expf(-g[1]);
            }
            *reinterpret_cast<__nv_bfloat162*>(a.out + t * a.out_st + h * a.out_sh + j) = __floats2bfloat162_rn(u, v);
        }
    }
}

// Whether the tensor-core form takes these operands: 16-byte loads along each operand's contiguous direction, paired stores.
static bool head_project_mma_takes(const void* in, int in_dtype, long long in_st, long long in_sh, const void* w, long long w_sh,
                                   long long w_sd, long long w_sj, const void* out, long long out_st, long long out_sh, int n_in,
                                   int n_out) {
    const int in_pack = in_dtype == MLC_DTYPE_F32 ? 4 : 8;
    const bool by_d = w_sd == 1;
    if (!by_d && w_sj != 1) return false;
    const long long w_ld = by_d ? w_sj : w_sd;
    if (n_in % 8 != 0 || (by_d ? n_out % 2 : n_out % 8) != 0) return false;
    if (w_ld % 8 != 0 || w_sh % 8 != 0 || in_st % in_pack != 0 || in_sh % in_pack != 0 || out_st % 2 != 0 || out_sh % 2 != 0) return false;
    return ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(w)) & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 3) == 0;
}

template <typename TI>
static cudaError_t launch_head_project_mma(const HeadProjectArgs& a, bool by_d, int H, cudaStream_t s) {
    const int tm = a.n <= 16 ? 16 : 64;
    const dim3 grid((a.n_out + 63) / 64, (a.n + tm - 1) / tm, H), block(128);
    if (tm == 16) return launch_pdl(by_d ? head_project_mma_kernel<TI, 16, true> : head_project_mma_kernel<TI, 16, false>, grid, block, 0, s, a);
    return launch_pdl(by_d ? head_project_mma_kernel<TI, 64, true> : head_project_mma_kernel<TI, 64, false>, grid, block, 0, s, a);
}

}  // namespace mlc

using namespace mlc;

extern "C" int mlc_latent_prepare(const float* proj, long long stride, const float* qsrc, long long q_stride, int interleaved,
                                  int q_col, int kv_col, const float* gain, float eps,
                                  const int* positions, const int* tok_seq, const void* rope_table, int rope_positions, int n,
                                  int H, int dim, int rot, int rank, int D, void* q_out, int dtype, int write_cache,
                                  void* k_pool, const int* page_table, long long entry_offset, int pages_per_seq,
                                  int page_size, void* stream) {
    if (n <= 0) return 0;
    if (H <= 0 || dim < 0 || rot < 0 || (rot & 1) || rank <= 0 || D < rank + rot || (write_cache && gain == nullptr)) return MLC_ERR_BAD_SIZE;
    PagedKV c{k_pool, k_pool, page_table, entry_offset, pages_per_seq, page_size, 1, D};
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = 32 * (H + 1 < 8 ? H + 1 : 8);
    if (dtype == MLC_DTYPE_F32)
        latent_prepare_kernel<float><<<n, threads, 0, s>>>(proj, stride, qsrc, q_stride, interleaved, q_col, kv_col, gain, eps, positions, tok_seq,
                                                           (const float2*)rope_table, rope_positions, H, dim, rot, rank, D,
                                                           (float*)q_out, write_cache, c);
    else if (dtype == MLC_DTYPE_BF16)
        latent_prepare_kernel<bf16><<<n, threads, 0, s>>>(proj, stride, qsrc, q_stride, interleaved, q_col, kv_col, gain, eps, positions, tok_seq,
                                                          (const float2*)rope_table, rope_positions, H, dim, rot, rank, D,
                                                          (bf16*)q_out, write_cache, c);
    else
        return MLC_ERR_BAD_DTYPE;
    MLC_LAUNCH_CHECK();
    return 0;
}

extern "C" int mlc_head_project(const void* in, int in_dtype, long long in_st, long long in_sh, const void* w, int w_dtype,
                                long long w_sh, long long w_sd, long long w_sj, void* out, int out_dtype, long long out_st,
                                long long out_sh, int n, int H, int n_in, int n_out, const float* gate, long long gate_st,
                                void* stream) {
    if (n <= 0) return 0;
    if (H <= 0 || H > 65535 || n_in <= 0 || n_out <= 0) return MLC_ERR_BAD_SIZE;
    const dim3 grid((n_out + HP_TILE - 1) / HP_TILE, (n + HP_TILE - 1) / HP_TILE, H);
    if (grid.y > 65535) return MLC_ERR_BAD_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    if (w_dtype == MLC_DTYPE_BF16 && out_dtype == MLC_DTYPE_BF16 &&
        head_project_mma_takes(in, in_dtype, in_st, in_sh, w, w_sh, w_sd, w_sj, out, out_st, out_sh, n_in, n_out)) {
        const bool by_d = w_sd == 1;
        const HeadProjectArgs a{in, in_st, in_sh, (const bf16*)w, w_sh, by_d ? w_sj : w_sd, (bf16*)out, out_st, out_sh, n, n_in,
                                n_out, gate, gate_st};
        const cudaError_t e = in_dtype == MLC_DTYPE_F32 ? launch_head_project_mma<float>(a, by_d, H, s)
                                                        : launch_head_project_mma<bf16>(a, by_d, H, s);
        return e == cudaSuccess ? 0 : (int)e;
    }
    const int code = in_dtype * 4 + w_dtype * 2 + out_dtype;
#define MLC_HP(TI, TW, TO)                                                                                                  \
    head_project_kernel<TI, TW, TO><<<grid, 256, 0, s>>>((const TI*)in, in_st, in_sh, (const TW*)w, w_sh, w_sd, w_sj, (TO*)out, \
                                                         out_st, out_sh, n, n_in, n_out, gate, gate_st)
    switch (code) {
        case 0: MLC_HP(float, float, float); break;
        case 1: MLC_HP(float, float, bf16); break;
        case 2: MLC_HP(float, bf16, float); break;
        case 3: MLC_HP(float, bf16, bf16); break;
        case 4: MLC_HP(bf16, float, float); break;
        case 5: MLC_HP(bf16, float, bf16); break;
        case 6: MLC_HP(bf16, bf16, float); break;
        case 7: MLC_HP(bf16, bf16, bf16); break;
        default: return MLC_ERR_BAD_DTYPE;
    }
#undef MLC_HP
    MLC_LAUNCH_CHECK();
    return 0;
}
