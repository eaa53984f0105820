// Kernels of the layered model family: decoders described layer by layer (ft_layer_desc), whose sizes are all run-time
// values.  The residual stream, the normed layer input, every projection output, attention scores and weights, router
// scores and the recurrent state are fp32; weights are bf16 and are multiplied as the fp32 numbers they are, with fp32
// accumulation in a fixed order per output element — a row's result does not depend on which other rows share its launch.
//
//   linear              C[r, n] = sum_k A[row(r), k] * W[p][n, k]: plain, batched over heads (column offsets per problem)
//                       or grouped over experts (row segments per problem, rows gathered through an index list), with
//                       fused epilogues (paired SwiGLU, tanh soft cap); a 64 x 64 tile kernel for many rows and a
//                       warp-per-output kernel for a handful of rows (decode)
//   embed / combine     embedding gather; gated-residual update of the stream, both fused with the scalar-gain RMS norm
//                       of the next layer
//   latent attention    the latent of every token is normed and written to a paged fp32 cache; queries are folded into
//                       latent space (q W_uk), scores, softmax and the weighted sum run over the cached latents, values
//                       are expanded afterwards (W_uv): only the latent is ever stored
//   channel delta       short causal convolutions + SiLU + unit norms + per-channel decays, then the gated delta rule
//                       token by token with one thread per state column, state and convolution tails in per-session slots
//   router              softmax over all experts, group-limited top-k, counting sort of (token, choice) pairs by expert
#include "common.cuh"
#include "ft_internal.h"

#include <algorithm>

namespace ft {

__device__ __forceinline__ float sigmoidf_(float x) { return 1.f / (1.f + __expf(-x)); }
__device__ __forceinline__ float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float bf16_to_f(const __nv_bfloat16* p) { return __bfloat162float(*p); }

__device__ __forceinline__ float block_sum(float v, float* red) {      // red: >= 33 floats of shared memory
    v = warp_sum(v);
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    __syncthreads();
    if (lane == 0) red[wid] = v;
    __syncthreads();
    if (wid == 0) {
        float t = lane < nw ? red[lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) red[32] = t;
    }
    __syncthreads();
    return red[32];
}

// asynchronous global -> shared copies (the staging of the delta rule and of the tensor-core attention)
__device__ __forceinline__ void cp_async4(float* dst_smem, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst_smem)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// ------------------------------------------------------------------ linear: tile kernel
constexpr int LBM = 64, LBN = 64, LBK = 16, LTHREADS = 256;

template <bool VEC>
__global__ void __launch_bounds__(LTHREADS) linear_tile_kernel(LinearArgs a) {
    __shared__ float sA[LBK][LBM + 4];
    __shared__ float sW[LBK][LBN + 4];
    __shared__ int s_info[3];
    int p, row0, rows_end;
    if (a.seg) {                       // grouped: blockIdx.y enumerates the row tiles of all segments
        if (threadIdx.x == 0) {
            int tile = blockIdx.y, pp = 0, found = -1, r0 = 0, r1 = 0;
            for (; pp < a.P; ++pp) {
                const int s0 = a.seg[pp], s1 = a.seg[pp + 1];
                const int nt = (s1 - s0 + LBM - 1) / LBM;
                if (tile < nt) { found = pp; r0 = s0 + tile * LBM; r1 = s1; break; }
                tile -= nt;
            }
            s_info[0] = found; s_info[1] = r0; s_info[2] = r1;
        }
        __syncthreads();
        p = s_info[0]; row0 = s_info[1]; rows_end = s_info[2];
        if (p < 0) return;
    } else {
        p = blockIdx.z; row0 = blockIdx.y * LBM; rows_end = a.M;
    }
    const int n0 = blockIdx.x * LBN;
    const float* A = a.A + (size_t)p * a.a_col_stride;
    const __nv_bfloat16* W = a.W + (size_t)p * a.w_stride;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;      // 16 x 16 threads, 4 x 4 outputs each
    // Every output is summed in two levels: the LBK products of a K tile in one short chain, the tiles' sums with a running
    // compensation term (the rounding error of each addition is carried into the next), so the result's error does not grow
    // with K as one long chain of multiply-adds would.
    float acc[4][4], comp[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = comp[i][j] = 0.f;
    // loader mapping: thread -> (row within tile, 4 consecutive k)
    const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
    const int arow_t = row0 + lr;
    long long arow = -1;
    if (arow_t < rows_end) arow = a.a_rows ? a.a_rows[arow_t] : arow_t;
    const int wrow = n0 + lr;
    for (int k0 = 0; k0 < a.K; k0 += LBK) {
        float av[4] = {0.f, 0.f, 0.f, 0.f}, wv[4] = {0.f, 0.f, 0.f, 0.f};
        const int k = k0 + lk;
        if (arow >= 0) {
            const float* ap = A + arow * a.lda + k;
            if (VEC && k + 3 < a.K) {
                const float4 t = *reinterpret_cast<const float4*>(ap);
                av[0] = t.x; av[1] = t.y; av[2] = t.z; av[3] = t.w;
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i) if (k + i < a.K) av[i] = ap[i];
            }
        }
        if (wrow < a.N) {
            const __nv_bfloat16* wp = W + (size_t)wrow * a.ldw + k;
            if (VEC && k + 3 < a.K) {
                const uint2 t = *reinterpret_cast<const uint2*>(wp);
                wv[0] = bf16_lo(t.x); wv[1] = bf16_hi(t.x); wv[2] = bf16_lo(t.y); wv[3] = bf16_hi(t.y);
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i) if (k + i < a.K) wv[i] = __bfloat162float(wp[i]);
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 4; ++i) { sA[lk + i][lr] = av[i]; sW[lk + i][lr] = wv[i]; }
        __syncthreads();
        float part[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) part[i][j] = 0.f;
#pragma unroll
        for (int kk = 0; kk < LBK; ++kk) {
            const float4 x = *reinterpret_cast<const float4*>(&sA[kk][ty * 4]);
            const float4 w = *reinterpret_cast<const float4*>(&sW[kk][tx * 4]);
            const float xa[4] = {x.x, x.y, x.z, x.w}, wa[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) part[i][j] = fmaf(xa[i], wa[j], part[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float y = part[i][j] - comp[i][j];
                const float t = __fadd_rn(acc[i][j], y);
                comp[i][j] = __fadd_rn(__fadd_rn(t, -acc[i][j]), -y);
                acc[i][j] = t;
            }
    }
    float* C = a.C + (size_t)p * a.c_col_stride;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = row0 + ty * 4 + i;
        if (r >= rows_end) continue;
        if (a.epi == LIN_SWIGLU_PAIR) {          // columns (2j, 2j+1) = (gate_j, up_j) -> C[r, j]
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int n = n0 + tx * 4 + j;
                if (n + 1 < a.N) C[(size_t)r * a.ldc + (n >> 1)] = glu_value(a.glu, acc[i][j], acc[i][j + 1], n >> 1);
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int n = n0 + tx * 4 + j;
                if (n < a.N) {
                    float v = acc[i][j];
                    if (a.epi == LIN_SOFTCAP) v = a.cap * tanhf(v / a.cap);
                    else if (a.epi == LIN_RELU2) { v = fmaxf(v, 0.f); v *= v; }
                    if (a.gate) v *= sigmoid_exact(a.gate[(size_t)r * a.ldg + (size_t)p * a.c_col_stride + n]);
                    if (a.C16) a.C16[(size_t)r * a.ldc + (size_t)p * a.c_col_stride + n] = __float2bfloat16_rn(v * a.c16_scale);
                    else C[(size_t)r * a.ldc + n] = v;
                }
            }
        }
    }
}

// ------------------------------------------------------------------ linear: few rows (decode)
// A CTA of 8 warps owns 32 output columns (16 column pairs with the SwiGLU epilogue) of one problem and walks its rows
// LROWS at a time: a slice of LKC columns of those rows is staged in shared memory once and reused by every column, each warp
// streams the weights of its columns 16 bytes per lane per load, so the weights are read once per LROWS rows.
// LROWS x LKC: 16 x 512, or 4 x 2048 where a problem has a handful of rows at most (more warps per SM, fewer barriers).
constexpr int LWARPS = 8, LROWS_MANY = 16, LROWS_FEW = 4, LSTAGE = 8192;

template <bool PAIR, bool VEC, int LROWS>
__global__ void __launch_bounds__(LWARPS * 32) linear_rows_kernel(LinearArgs a) {
    constexpr int LKC = LSTAGE / LROWS;
    constexpr int CPW = PAIR ? 2 : 4;                 // output columns per warp
    constexpr int WR = PAIR ? 2 * CPW : CPW;          // weight rows per warp
    __shared__ __align__(16) float sA[LROWS][LKC];
    const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int cols = PAIR ? a.N / 2 : a.N;
    const int p = blockIdx.y;
    const int col0 = (blockIdx.x * LWARPS + wid) * CPW;
    int r0 = 0, r1 = a.M;
    if (a.seg) { r0 = a.seg[p]; r1 = a.seg[p + 1]; }
    if (r1 <= r0) return;
    const float* A = a.A + (size_t)p * a.a_col_stride;
    const __nv_bfloat16* W = a.W + (size_t)p * a.w_stride;
    float* C = a.C + (size_t)p * a.c_col_stride;
    const __nv_bfloat16* wrow[WR];
    bool wok[WR];
#pragma unroll
    for (int c = 0; c < WR; ++c) {
        const int n = PAIR ? 2 * col0 + c : col0 + c;
        wok[c] = n < a.N;
        wrow[c] = W + (size_t)(wok[c] ? n : 0) * a.ldw;
    }
    for (int rb = r0; rb < r1; rb += LROWS) {
        const int nr = min(LROWS, r1 - rb);
        float acc[WR][LROWS];
#pragma unroll
        for (int c = 0; c < WR; ++c)
#pragma unroll
            for (int i = 0; i < LROWS; ++i) acc[c][i] = 0.f;
        for (int k0 = 0; k0 < a.K; k0 += LKC) {
            const int kc = min(LKC, a.K - k0);
            __syncthreads();
            for (int i = wid; i < nr; i += LWARPS) {          // a warp per row
                const int r = rb + i;
                const float* src = A + (size_t)(a.a_rows ? a.a_rows[r] : r) * a.lda + k0;
                if (VEC) {
                    for (int k = lane * 4; k < kc; k += 128)
                        *reinterpret_cast<float4*>(&sA[i][k]) = *reinterpret_cast<const float4*>(src + k);
                } else {
                    for (int k = lane; k < kc; k += 32) sA[i][k] = src[k];
                }
            }
            __syncthreads();
            if (VEC) {
                for (int k = lane * 8; k < kc; k += 256) {
                    float wv[WR][8];
#pragma unroll
                    for (int c = 0; c < WR; ++c) {
                        uint4 t = make_uint4(0u, 0u, 0u, 0u);
                        if (wok[c]) t = __ldg(reinterpret_cast<const uint4*>(wrow[c] + k0 + k));
                        wv[c][0] = bf16_lo(t.x); wv[c][1] = bf16_hi(t.x); wv[c][2] = bf16_lo(t.y); wv[c][3] = bf16_hi(t.y);
                        wv[c][4] = bf16_lo(t.z); wv[c][5] = bf16_hi(t.z); wv[c][6] = bf16_lo(t.w); wv[c][7] = bf16_hi(t.w);
                    }
#pragma unroll
                    for (int i = 0; i < LROWS; ++i) {
                        if (i < nr) {
                            const float4 x0 = *reinterpret_cast<const float4*>(&sA[i][k]);
                            const float4 x1 = *reinterpret_cast<const float4*>(&sA[i][k + 4]);
                            const float xa[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
                            for (int c = 0; c < WR; ++c)
#pragma unroll
                                for (int e = 0; e < 8; ++e) acc[c][i] = fmaf(xa[e], wv[c][e], acc[c][i]);
                        }
                    }
                }
            } else {
                for (int k = lane; k < kc; k += 32) {
                    float wv[WR];
#pragma unroll
                    for (int c = 0; c < WR; ++c) wv[c] = wok[c] ? __bfloat162float(wrow[c][k0 + k]) : 0.f;
#pragma unroll
                    for (int i = 0; i < LROWS; ++i)
                        if (i < nr) {
                            const float x = sA[i][k];
#pragma unroll
                            for (int c = 0; c < WR; ++c) acc[c][i] = fmaf(x, wv[c], acc[c][i]);
                        }
                }
            }
        }
#pragma unroll
        for (int c = 0; c < CPW; ++c) {
#pragma unroll
            for (int i = 0; i < LROWS; ++i) {
                if (i >= nr) continue;               // uniform over the warp
                float v;
                if (PAIR) {
                    const float g = warp_sum(acc[2 * c][i]), u = warp_sum(acc[2 * c + 1][i]);
                    v = lane == 0 && col0 + c < cols ? glu_value(a.glu, g, u, col0 + c) : 0.f;
                } else {
                    v = warp_sum(acc[c][i]);
                    if (a.epi == LIN_SOFTCAP) v = a.cap * tanhf(v / a.cap);
                    else if (a.epi == LIN_RELU2) { v = fmaxf(v, 0.f); v *= v; }
                    if (a.gate && lane == 0 && col0 + c < cols)
                        v *= sigmoid_exact(a.gate[(size_t)(rb + i) * a.ldg + (size_t)p * a.c_col_stride + col0 + c]);
                }
                if (lane == 0 && col0 + c < cols) {
                    if (a.C16) a.C16[(size_t)(rb + i) * a.ldc + (size_t)p * a.c_col_stride + col0 + c] = __float2bfloat16_rn(v * a.c16_scale);
                    else C[(size_t)(rb + i) * a.ldc + col0 + c] = v;
                }
            }
        }
    }
}

int launch_linear(const LinearArgs& a, int rows_bound, cudaStream_t stream) {
    if (rows_bound <= 0 || a.N <= 0) return 0;
    FT_REQUIRE(a.K >= 1 && a.P >= 1, "linear: bad sizes");
    FT_REQUIRE(a.epi != LIN_SWIGLU_PAIR || (a.N & 1) == 0, "linear: the paired epilogue needs an even number of rows");
    // few rows per problem: one warp per output column, the weights stream once
    const bool few = a.seg ? rows_bound <= 4 * LROWS_MANY : rows_bound <= 2 * LROWS_MANY;
    if (few) {
        const bool pair = a.epi == LIN_SWIGLU_PAIR;
        const int cols = pair ? a.N / 2 : a.N;
        const int per_cta = LWARPS * (pair ? 2 : 4);
        const bool v8 = (a.K & 7) == 0 && (a.ldw & 7) == 0 && (a.lda & 3) == 0 && (a.a_col_stride & 3) == 0 &&
                        (a.w_stride & 7) == 0 && ((uintptr_t)a.A & 15) == 0 && ((uintptr_t)a.W & 15) == 0;
        dim3 grid((cols + per_cta - 1) / per_cta, a.P);
        // rows per problem: M, or about rows_bound / P of a grouped launch
        const bool handful = a.seg ? rows_bound <= 3 * a.P : a.M <= LROWS_FEW;
#define FT_ROWS(PAIR_, VEC_)                                                                                             \
    do {                                                                                                                 \
        if (handful) linear_rows_kernel<PAIR_, VEC_, LROWS_FEW><<<grid, LWARPS * 32, 0, stream>>>(a);                    \
        else linear_rows_kernel<PAIR_, VEC_, LROWS_MANY><<<grid, LWARPS * 32, 0, stream>>>(a);                           \
    } while (0)
        if (pair) {
            if (v8) FT_ROWS(true, true);
            else FT_ROWS(true, false);
        } else {
            if (v8) FT_ROWS(false, true);
            else FT_ROWS(false, false);
        }
#undef FT_ROWS
        FT_CHECK_CUDA(cudaGetLastError());
        return 0;
    }
    const bool vec = (a.lda & 3) == 0 && (a.ldw & 3) == 0 && (a.a_col_stride & 3) == 0 && (a.w_stride & 3) == 0 &&
                     ((uintptr_t)a.A & 15) == 0 && ((uintptr_t)a.W & 7) == 0;
    dim3 grid((a.N + LBN - 1) / LBN, 1, 1);
    if (a.seg) grid.y = (rows_bound + LBM - 1) / LBM + a.P;
    else { grid.y = (a.M + LBM - 1) / LBM; grid.z = a.P; }
    if (vec) linear_tile_kernel<true><<<grid, LTHREADS, 0, stream>>>(a);
    else linear_tile_kernel<false><<<grid, LTHREADS, 0, stream>>>(a);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

// ------------------------------------------------------------------ bf16 planes for the tensor-core projections
// v = hi + lo with hi = bf16(v), lo = bf16(v - hi): the tcgen05 GEMM multiplies both planes into one fp32 accumulator, which
// keeps about 16 mantissa bits of an fp32 activation.
__device__ __forceinline__ void store_planes(__nv_bfloat16* hi, __nv_bfloat16* lo, size_t i, float v) {
    const __nv_bfloat16 h = __float2bfloat16_rn(v);
    hi[i] = h;
    lo[i] = __float2bfloat16_rn(v - __bfloat162float(h));
}

__global__ void to_planes_kernel(const float* __restrict__ x, __nv_bfloat16* __restrict__ hi, __nv_bfloat16* __restrict__ lo,
                                 size_t n) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        store_planes(hi, lo, i, x[i]);
}

__global__ void softcap_kernel(float* __restrict__ x, size_t n, float cap) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] / cap);
}

// planes of the rows an index list names: out row i = planes(src[idx[i]])
__global__ void gather_planes_kernel2(const float* __restrict__ src, const int* __restrict__ idx, __nv_bfloat16* __restrict__ hi,
                                      __nv_bfloat16* __restrict__ lo, int W) {
    const size_t i = blockIdx.x;
    const float* r = src + (size_t)idx[i] * W;
    for (int c = threadIdx.x; c < W; c += blockDim.x) store_planes(hi, lo, i * W + c, r[c]);
}

// gu [rows][2 ff] with columns (2j, 2j+1) = (gate_j, up_j)  ->  planes of their gated product (GluSpec), [rows][ff]
__global__ void glu_planes_kernel(const float* __restrict__ gu, __nv_bfloat16* __restrict__ hi, __nv_bfloat16* __restrict__ lo, size_t n,
                                  int ff, GluSpec glu) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const float2 v = reinterpret_cast<const float2*>(gu)[i];
        store_planes(hi, lo, i, glu_value(glu, v.x, v.y, glu.bias ? (int)(i % ff) : 0));
    }
}

// u [rows][ff]  ->  planes of relu(u)^2
__global__ void relu2_planes_kernel(const float* __restrict__ u, __nv_bfloat16* __restrict__ hi, __nv_bfloat16* __restrict__ lo,
                                    size_t n) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const float v = fmaxf(u[i], 0.f);
        store_planes(hi, lo, i, v * v);
    }
}

int launch_gather_planes_rows(const float* src, const int* idx, void* hi, void* lo, int n, int W, cudaStream_t stream) {
    gather_planes_kernel2<<<n, 256, 0, stream>>>(src, idx, (__nv_bfloat16*)hi, (__nv_bfloat16*)lo, W);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}
int launch_act_planes(const float* gu, void* hi, void* lo, int rows, int ff, int act, const GluSpec& glu, cudaStream_t stream) {
    const size_t n = (size_t)rows * ff;
    const int blocks = (int)std::min<size_t>((n + 255) / 256, 148 * 16);
    if (act == FT_ACT_RELU2) relu2_planes_kernel<<<blocks, 256, 0, stream>>>(gu, (__nv_bfloat16*)hi, (__nv_bfloat16*)lo, n);
    else glu_planes_kernel<<<blocks, 256, 0, stream>>>(gu, (__nv_bfloat16*)hi, (__nv_bfloat16*)lo, n, ff, glu);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

int launch_to_planes(const float* x, void* hi, void* lo, size_t n, cudaStream_t stream) {
    const int blocks = (int)std::min<size_t>((n + 255) / 256, 148 * 16);
    to_planes_kernel<<<blocks, 256, 0, stream>>>(x, (__nv_bfloat16*)hi, (__nv_bfloat16*)lo, n);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}
int launch_softcap(float* x, size_t n, float cap, cudaStream_t stream) {
    const int blocks = (int)std::min<size_t>((n + 255) / 256, 148 * 16);
    softcap_kernel<<<blocks, 256, 0, stream>>>(x, n, cap);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

// ------------------------------------------------------------------ embedding / residual update, fused with the next norm
// hn[t] = x[t] / sqrt(mean(x[t]^2) + eps) * gain, the gain being one number.
__global__ void __launch_bounds__(256)
embed_norm_kernel(const int* __restrict__ tokens, const __nv_bfloat16* __restrict__ embed, float* __restrict__ x,
                  float* __restrict__ hn, __nv_bfloat16* __restrict__ hi, __nv_bfloat16* __restrict__ lo, int W, float eps,
                  float gain, const float* __restrict__ gain_w) {
    __shared__ float red[33];
    const int t = blockIdx.x;
    const __nv_bfloat16* e = embed + (size_t)tokens[t] * W;
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        const float v = __bfloat162float(e[c]);
        x[(size_t)t * W + c] = v;
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float r = gain / sqrtf(ss / (float)W + eps);
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        float v = __bfloat162float(e[c]) * r;
        if (gain_w) v *= gain_w[c];
        hn[(size_t)t * W + c] = v;
        if (hi) store_planes(hi, lo, (size_t)t * W + c, v);
    }
}

// x[t] += sigmoid(rg1[t] + b1) * mix[t] + sigmoid(rg2[t] + b2) * sum_k wt[t, k] * eout[slot_pos[t, k]]   (feed-forward
// part only when top > 0), then the next norm of the row.  rg1 / rg2 are column ranges of the input projection `proj`.
__global__ void __launch_bounds__(256)
combine_norm_kernel(float* __restrict__ x, float* __restrict__ hn, const float* __restrict__ proj, int ldp, int o_rg1,
                    int o_rg2, const float* __restrict__ rg_bias, const float* __restrict__ mix,
                    const float* __restrict__ eout, const float* __restrict__ wt, const int* __restrict__ slot_pos,
                    int top, int W, float eps, float gain, __nv_bfloat16* __restrict__ hi, __nv_bfloat16* __restrict__ lo) {
    __shared__ float red[33];
    extern __shared__ float row[];
    const int t = blockIdx.x;
    const float* pr = proj + (size_t)t * ldp;
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        float y = sigmoid_exact(pr[o_rg1 + c] + rg_bias[c]) * mix[(size_t)t * W + c];
        if (top > 0) {
            float f = 0.f;
            for (int k = 0; k < top; ++k)
                f = fmaf(wt[(size_t)t * top + k], eout[(size_t)slot_pos[(size_t)t * top + k] * W + c], f);
            y += sigmoid_exact(pr[o_rg2 + c] + rg_bias[W + c]) * f;
        }
        const float v = x[(size_t)t * W + c] + y;
        x[(size_t)t * W + c] = v;
        row[c] = v;
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float r = gain / sqrtf(ss / (float)W + eps);
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        const float v = row[c] * r;
        hn[(size_t)t * W + c] = v;
        if (hi) store_planes(hi, lo, (size_t)t * W + c, v);
    }
}

// rows of the normed stream that the head reads: out[i] = hn[idx[i]]
__global__ void gather_rows_kernel(const float* __restrict__ src, const int* __restrict__ idx, float* __restrict__ dst, int W) {
    const int i = blockIdx.x;
    const float* s = src + (size_t)idx[i] * W;
    for (int c = threadIdx.x; c < W; c += blockDim.x) dst[(size_t)i * W + c] = s[c];
}

int launch_embed_norm(const int* tokens, const void* embed, float* x, float* hn, void* hi, void* lo, int T, int W, float eps,
                      float gain, const float* gain_w, cudaStream_t stream) {
    embed_norm_kernel<<<T, 256, 0, stream>>>(tokens, (const __nv_bfloat16*)embed, x, hn, (__nv_bfloat16*)hi, (__nv_bfloat16*)lo,
                                             W, eps, gain_w ? 1.f : gain, gain_w);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}
int launch_combine_norm(float* x, float* hn, const float* proj, int ldp, int o_rg1, int o_rg2, const float* rg_bias,
                        const float* mix, const float* eout, const float* wt, const int* slot_pos, int top, int T, int W,
                        float eps, float gain, void* hi, void* lo, cudaStream_t stream) {
    combine_norm_kernel<<<T, 256, (size_t)W * 4, stream>>>(x, hn, proj, ldp, o_rg1, o_rg2, rg_bias, mix, eout, wt, slot_pos,
                                                          top, W, eps, gain, (__nv_bfloat16*)hi, (__nv_bfloat16*)lo);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}
int launch_gather_rows(const float* src, const int* idx, float* dst, int n, int W, cudaStream_t stream) {
    gather_rows_kernel<<<n, 256, 0, stream>>>(src, idx, dst, W);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

// ------------------------------------------------------------------ latent attention
// Token t: c = raw / sqrt(mean(raw^2) + eps) * w and the rotated shared key part go to page_table[seq_rows[t]][pos / 64], row
// pos % 64 of the layer's caches ([page][64][rank + rot] fp32; bf16 as latent_chunk16 lays a page out); the rotated part
// of every query head goes to qlat.  Pairs (i, i + rot / 2); the angle's sine and cosine are formed once per token.
__global__ void __launch_bounds__(128) latent_prep_kernel(LatentArgs a, int row16) {
    __shared__ float red[33];
    extern __shared__ float trig[];                        // [rot / 2] cosines, [rot / 2] sines
    const int t = blockIdx.x, rank = a.rank, rot = a.rot, half = rot >> 1;
    const float* pr = a.proj + (size_t)t * a.ldp;
    const float* raw = pr + a.o_dkv;
    const int pos = a.positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf((float)pos * a.rot_freq[i], &trig[half + i], &trig[i]);
    float ss = 0.f;
    for (int c = threadIdx.x; c < rank; c += blockDim.x) ss += raw[c] * raw[c];
    ss = block_sum(ss, red);                               // its barriers also publish trig
    const float r = 1.f / sqrtf(ss / (float)rank + a.eps);
    const int page = a.page_table[(size_t)a.seq_rows[t] * a.max_pages + pos / kKvTile];
    const int slot = pos % kKvTile;
    float* c32 = a.cache ? a.cache + ((size_t)page * kKvTile + slot) * (rank + rot) : nullptr;
    __nv_bfloat16* c16 = a.cache16 ? (__nv_bfloat16*)a.cache16 + (size_t)page * kKvTile * row16 : nullptr;
    auto at16 = [&](int c) { return latent_chunk16(slot, c >> 3) + (c & 7); };
    for (int c = threadIdx.x; c < rank; c += blockDim.x) {
        const float v = raw[c] * r * a.norm_w[c];
        if (c32) c32[c] = v;
        if (c16) c16[at16(c)] = __float2bfloat16_rn(v);
    }
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float u = raw[rank + i], v = raw[rank + half + i], cs = trig[i], sn = trig[half + i];
        const float x = u * cs - v * sn, y = v * cs + u * sn;
        if (c32) { c32[rank + i] = x; c32[rank + half + i] = y; }
        if (c16) { c16[at16(rank + i)] = __float2bfloat16_rn(x); c16[at16(rank + half + i)] = __float2bfloat16_rn(y); }
    }
    const int hd = a.dim + rot, kd = rank + rot;
    for (int j = threadIdx.x; j < a.H * half; j += blockDim.x) {
        const int h = j / half, i = j % half;
        const float* q = pr + a.o_q + h * hd + a.dim;
        const float u = q[i], v = q[half + i], cs = trig[i], sn = trig[half + i];
        const float x = u * cs - v * sn, y = v * cs + u * sn;
        if (a.qlat16) {
            __nv_bfloat16* dst = a.qlat16 + ((size_t)t * a.H + h) * row16 + rank;
            dst[i] = __float2bfloat16_rn(x * a.scale);
            dst[half + i] = __float2bfloat16_rn(y * a.scale);
        } else {
            float* dst = a.qlat + ((size_t)t * a.H + h) * kd + rank;
            dst[i] = x;
            dst[half + i] = y;
        }
    }
    if (a.qlat16 && kd < row16)
        for (int j = threadIdx.x; j < a.H * (row16 - kd); j += blockDim.x)
            a.qlat16[((size_t)t * a.H + j / (row16 - kd)) * row16 + kd + j % (row16 - kd)] = __float2bfloat16_rn(0.f);
}

// One warp per (token, head, key range): the query in latent space stays in registers (NR values per lane), keys = values =
// the cached latents, online softmax in fp32.  Keys are taken KB at a time: their rows are all requested before the first
// is used and the KB score reductions interleave, so the loop waits for memory once per block instead of once per key.
// With n_split == 1 the warp finishes its (token, head): divides by the softmax sum and scales by the head's output gate
// sigmoid(gate logit) — the value expansion that follows is linear, so gating before it is the same.  With n_split > 1
// (few tokens: decode) it covers the s-th share of the keys and leaves (max, sum, unnormalised result) for the merge.
// The softmax sum of a row whose maximum is m, with the sink's term, and the factor that finishes the row's result.
__device__ __forceinline__ float latent_finish(float m, float l, const LatentArgs& a, int t, int h) {
    float g = 1.f;
    if (a.sink) {
        // relative to the larger of m and the sink, so that neither exponential overflows
        const float s = a.sink[h], top = fmaxf(m, s);
        const float f = expf(m - top);
        g = f;
        l = l * f + expf(s - top);
    }
    if (a.o_gate >= 0) g *= sigmoid_exact(a.proj[(size_t)t * a.ldp + a.o_gate + h]);
    return g / l;
}

template <int NR, int KB>
__global__ void __launch_bounds__(128) latent_attn_kernel(LatentArgs a, int n_pairs, int n_split) {
    const int pair = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    const int split = blockIdx.y;
    if (pair >= n_pairs) return;
    const int rank = a.rank, kd = a.rank + a.rot;
    const int t = pair / a.H, h = pair % a.H;
    const float* cache = a.cache;
    const float* q = a.qlat + (size_t)pair * kd;
    float qr[NR], acc[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int c = lane + 32 * i;
        qr[i] = c < kd ? q[c] * a.scale : 0.f;
        acc[i] = 0.f;
    }
    const int n_keys = a.positions[t] + 1;
    int j_lo = 0, j_hi = n_keys;
    if (n_split > 1) {          // shares of whole pages
        const int share = ((n_keys + n_split - 1) / n_split + kKvTile - 1) / kKvTile * kKvTile;
        j_lo = min(split * share, n_keys);
        j_hi = min(j_lo + share, n_keys);
    }
    const int* pt = a.page_table + (size_t)a.seq_rows[t] * a.max_pages;
    float m = -INFINITY, l = 0.f;
    for (int j0 = j_lo; j0 < j_hi; j0 += KB) {
        float cv[KB][NR], sc[KB];
#pragma unroll
        for (int b = 0; b < KB; ++b) {
            const int j = min(j0 + b, j_hi - 1);
            const float* c = cache + ((size_t)pt[j / kKvTile] * kKvTile + j % kKvTile) * kd;
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const int cc = lane + 32 * i;
                cv[b][i] = cc < kd ? c[cc] : 0.f;
            }
        }
#pragma unroll
        for (int b = 0; b < KB; ++b) {
            float x = 0.f;
#pragma unroll
            for (int i = 0; i < NR; ++i) x = fmaf(qr[i], cv[b][i], x);
            sc[b] = x;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int b = 0; b < KB; ++b) sc[b] += __shfl_xor_sync(0xffffffffu, sc[b], o);
        float mn = m;
#pragma unroll
        for (int b = 0; b < KB; ++b) {
            if (j0 + b >= j_hi) sc[b] = -INFINITY;
            mn = fmaxf(mn, sc[b]);
        }
        const float corr = expf(m - mn);
        l *= corr;
#pragma unroll
        for (int i = 0; i < NR; ++i) acc[i] *= corr;
#pragma unroll
        for (int b = 0; b < KB; ++b) {
            const float pw = expf(sc[b] - mn);          // 0 for the padding of the last block
            l += pw;
#pragma unroll
            for (int i = 0; i < NR; ++i) acc[i] = fmaf(pw, cv[b][i], acc[i]);
        }
        m = mn;
    }
    if (n_split > 1) {
        float* p = a.part + ((size_t)pair * n_split + split) * (rank + 2);
        if (lane == 0) { p[0] = m; p[1] = l; }
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int c = lane + 32 * i;
            if (c < rank) p[2 + c] = acc[i];
        }
        return;
    }
    const float g = latent_finish(m, l, a, t, h);
    float* o = a.out + (size_t)pair * rank;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int c = lane + 32 * i;
        if (c < rank) o[c] = acc[i] * g;
    }
}

int launch_latent_prep(const LatentArgs& a, int T, cudaStream_t stream) {
    FT_REQUIRE(a.proj && a.norm_w && (a.cache || a.cache16) && (a.rot == 0 || (a.rot_freq && (a.qlat || a.qlat16) && a.rot % 2 == 0)),
               "latent prep: missing operands");
    latent_prep_kernel<<<T, 128, (size_t)a.rot * 4, stream>>>(a, latent_row16(a.rank, a.rot));
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

int latent_row16(int rank, int rot) { return (rank + rot + 63) / 64 * 64; }
// the serving form keeps latents of whole 32-column pieces in bf16; other sizes stay in fp32 on the CUDA cores
bool latent_attn_mma_ok(int rank, int rot) { 
    LatentArgs one;
    one.H = 1;
    return rank >= 32 && rank % 32 == 0 && paged16_mma_ok(latent_paged(one, rank, rot));
}

// The latent cache as a paged bf16 cache: one key row for all heads, whose first columns are also the value.
Paged16Args latent_paged(const LatentArgs& a, int rank, int rot) {
    Paged16Args p;
    p.q = a.qlat16; p.cache = a.cache16; p.positions = a.positions; p.seq_rows = a.seq_rows; p.page_table = a.page_table;
    p.max_pages = a.max_pages; p.H = a.H; p.G = 1; p.key_blocks = p.blocks = latent_row16(rank, rot) / 64; p.v_block = 0; p.dim = rank + rot;
    p.vdim = rank; p.sink = a.sink; p.out = a.out; p.part = a.part;
    if (a.o_gate >= 0) { p.gate = a.proj + a.o_gate; p.ldg = a.ldp; }
    return p;
}

int launch_latent_attn(const LatentArgs& a, int T, cudaStream_t stream) {
    const int n_pairs = T * a.H;
    const int n_split = a.part ? attn_splits(T, a.H) : 1;
    if (a.cache16 && latent_attn_mma_ok(a.rank, a.rot)) {
        FT_REQUIRE(a.qlat16, "latent attention: no bf16 queries");
        return launch_paged16_mma(latent_paged(a, a.rank, a.rot), T, stream);
    } else {
        FT_REQUIRE(a.cache && a.qlat, "latent attention: no fp32 cache or queries");
        const int kd = a.rank + a.rot;
        const dim3 grid((n_pairs + 3) / 4, n_split);
#define FT_LAT(NR_, KB_) latent_attn_kernel<NR_, KB_><<<grid, 128, 0, stream>>>(a, n_pairs, n_split)
        if (kd <= 32) FT_LAT(1, 8);
        else if (kd <= 64) FT_LAT(2, 8);
        else if (kd <= 128) FT_LAT(4, 8);
        else if (kd <= 256) FT_LAT(8, 4);
        else if (kd <= 512) FT_LAT(16, 4);
        else { FT_REQUIRE(kd <= 1024, "latent attention: a cache row of %d columns is beyond 1024", kd); FT_LAT(32, 2); }
#undef FT_LAT
    }
    FT_CHECK_CUDA(cudaGetLastError());
    if (n_split > 1) {
        return launch_paged16_merge(latent_paged(a, a.rank, a.rot), n_pairs, n_split, stream);
    }
    return 0;
}

// ------------------------------------------------------------------ channel delta
// Per token: the three short convolutions over time + SiLU (inputs before the step's first token come from the session's
// tail of raw inputs; zeros before position 0), unit norms of q and k per head (q also times dim^-1/2), the decay
// exp(-exp(A_log_h) * softplus(a + dt_bias)) per head and key channel, beta = sigmoid.
// qkv out: [T][channels] with channels = 2 * kvh * dim + heads * vdim in the order q | k | v.
__global__ void __launch_bounds__(256)
delta_prep_kernel(DeltaArgs a) {
    extern __shared__ float sh[];
    const int t = blockIdx.x;
    const int req = a.seq_rows[t];
    const int r = t - a.req_start[req];              // index inside this step's portion
    const int pos0 = a.req_pos0[req];
    const int qk = a.kvh * a.dim, ch = 2 * qk + a.heads * a.vdim;
    const float* tail = a.state + (size_t)a.req_slot[req] * a.slot_stride + a.tail_off;
    const int taps = a.taps;
    for (int c = threadIdx.x; c < ch; c += blockDim.x) {
        float s = 0.f;
        for (int i = 0; i < taps; ++i) {
            const int back = taps - 1 - i;
            float v;
            if (r - back >= 0) v = a.proj[(size_t)(t - back) * a.ldp + a.o_q + c];
            else if (pos0 + r - back >= 0) v = tail[(size_t)c * (taps - 1) + (taps - 1 + r - back)];
            else v = 0.f;
            s = fmaf(a.conv[(size_t)c * taps + i], v, s);
        }
        sh[c] = s / (1.f + expf(-s));
    }
    __syncthreads();
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    float* dst = a.qkv + (size_t)t * ch;
    for (int hh = wid; hh < 2 * a.kvh; hh += nw) {          // q heads, then k heads
        const float* v = sh + (size_t)hh * a.dim;
        float ss = 0.f;
        for (int d = lane; d < a.dim; d += 32) ss += v[d] * v[d];
        ss = warp_sum(ss);
        float sc = 1.f / sqrtf(ss + 1e-6f);
        if (hh < a.kvh) sc *= 1.f / sqrtf((float)a.dim);
        for (int d = lane; d < a.dim; d += 32) dst[(size_t)hh * a.dim + d] = v[d] * sc;
    }
    for (int c = 2 * qk + threadIdx.x; c < ch; c += blockDim.x) dst[c] = sh[c];
    const int hd = a.heads * a.dim;
    for (int i = threadIdx.x; i < hd; i += blockDim.x) {
        // one decay per head and key channel, or (head_decay) one per head, written to all of the head's channels
        const float z = a.head_decay ? a.araw[(size_t)t * a.ld_araw + i / a.dim] + a.dt_bias[i / a.dim]
                                     : a.araw[(size_t)t * hd + i] + a.dt_bias[i];
        const float sp = z > 20.f ? z : log1pf(expf(z));
        a.decay[(size_t)t * hd + i] = expf(-expf(a.a_log[i / a.dim]) * sp);
    }
    for (int h = threadIdx.x; h < a.heads; h += blockDim.x)
        a.beta[(size_t)t * a.heads + h] = sigmoid_exact(a.proj[(size_t)t * a.ldp + a.o_beta + h]);
}

// New tail of raw convolution inputs per (request, channel): the last taps-1 entries of (old tail ++ this step's inputs).
__global__ void delta_tail_kernel(DeltaArgs a, int n_req) {
    const int req = blockIdx.y;
    const int ch = 2 * a.kvh * a.dim + a.heads * a.vdim;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= ch || req >= n_req) return;
    const int n = a.req_start[req + 1] - a.req_start[req], pos0 = a.req_pos0[req], keep = a.taps - 1;
    float* tail = a.state + (size_t)a.req_slot[req] * a.slot_stride + a.tail_off + (size_t)c * keep;
    float v[16];
    for (int i = 0; i < keep; ++i) {
        const int src = n + i;                      // index into old tail (keep entries) ++ inputs (n entries)
        if (src < keep) v[i] = pos0 > 0 ? tail[src] : 0.f;
        else v[i] = a.proj[(size_t)(a.req_start[req] + src - keep) * a.ldp + a.o_q + c];
    }
    for (int i = 0; i < keep; ++i) tail[i] = v[i];
}

// The recurrence, one CTA per (request, head, block of DCOLS state columns).  Per token
//   S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// is local to a column of the state S [dim][vdim].  Four neighbouring lanes share a column, each holding a run of DPT key
// channels of it in registers, so the two sums over key channels are two short chains plus two shuffles.
// q, k, g, v, beta of DCHUNK tokens at a time are copied into shared memory asynchronously (cp.async), one chunk ahead
// of the one being computed.
constexpr int DCHUNK = 8, DCOLS = 32;

// Shared-memory layout of one staged token: q, k, g each as four runs of DPT channels (one per lane of a column's quad)
// with four floats of padding between runs, so that the quad's 16-byte reads fall into different banks; then v, then beta.
template <int DPT>
__host__ __device__ constexpr int delta_run() { return DPT + 4; }
__host__ __device__ inline int delta_token_floats(int dpt, int vdim) { return (12 * (dpt + 4) + vdim + 1 + 3) & ~3; }

// FULL: dim == 4 * DPT, every channel test is true at compile time (the tests otherwise compile to branches in the token loop).
template <int DPT, int MAXT, bool FULL>
__global__ void __launch_bounds__(MAXT)
delta_rule_kernel(DeltaArgs a) {
    extern __shared__ __align__(16) float sh[];
    constexpr int RUN = delta_run<DPT>();
    const int req = blockIdx.x, h = blockIdx.y;
    const int j = blockIdx.z * DCOLS + (threadIdx.x >> 2), part = threadIdx.x & 3;      // column, and which run of key channels
    const int kh = h / (a.heads / a.kvh);
    const int row0 = a.req_start[req], n = a.req_start[req + 1] - row0;
    const int dim = a.dim, vdim = a.vdim;
    const int qk = a.kvh * dim, ch = 2 * qk + a.heads * vdim, hd = a.heads * dim;
    float* S = a.state + (size_t)a.req_slot[req] * a.slot_stride + a.s_off + (size_t)h * dim * vdim;
    const bool live = j < vdim;
    const bool fresh = a.req_pos0[req] == 0;
    const int d0 = part * DPT;                    // this lane's channels: d0 .. d0 + DPT - 1
    float s[DPT];
#pragma unroll
    for (int i = 0; i < DPT; ++i) s[i] = (live && !fresh && d0 + i < dim) ? S[(size_t)(d0 + i) * vdim + j] : 0.f;
    const int per = delta_token_floats(DPT, vdim);
    const int o_k = 4 * RUN, o_g = 8 * RUN, o_v = 12 * RUN;
    const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    auto stage = [&](int c0, float* buf) {
        const int nc = min(DCHUNK, n - c0);
        for (int tt = wid; tt < nc; tt += nw) {          // a warp per token
            const size_t t = row0 + c0 + tt;
            float* dst = buf + (size_t)tt * per;
            const float* q = a.qkv + t * ch + (size_t)kh * dim;
            const float* g = a.decay + t * hd + (size_t)h * dim;
            const float* v = a.qkv + t * ch + 2 * qk + (size_t)h * vdim;
            for (int e = lane; e < dim; e += 32) {
                const int at = (e / DPT) * RUN + e % DPT;
                cp_async4(dst + at, q + e);
                cp_async4(dst + o_k + at, q + qk + e);
                cp_async4(dst + o_g + at, g + e);
            }
            for (int e = lane; e < vdim; e += 32) cp_async4(dst + o_v + e, v + e);
            if (lane == 0) cp_async4(dst + o_v + vdim, a.beta + t * a.heads + h);
        }
        cp_async_commit();
    };
    float* buf0 = sh;
    float* buf1 = sh + (size_t)DCHUNK * per;
    stage(0, buf0);
    for (int c0 = 0, it = 0; c0 < n; c0 += DCHUNK, ++it) {
        float* cur = (it & 1) ? buf1 : buf0;
        cp_async_wait_all();
        __syncthreads();                                  // chunk `it` has landed; everyone is done with the other buffer
        if (c0 + DCHUNK < n) stage(c0 + DCHUNK, (it & 1) ? buf0 : buf1);
        const int nc = min(DCHUNK, n - c0);
        for (int tt = 0; tt < nc; ++tt) {
            const float* base = cur + (size_t)tt * per;
            const float4* q4 = reinterpret_cast<const float4*>(base + part * RUN);
            const float4* k4 = reinterpret_cast<const float4*>(base + o_k + part * RUN);
            const float4* g4 = reinterpret_cast<const float4*>(base + o_g + part * RUN);
            float dot0 = 0.f, dot1 = 0.f;
#pragma unroll
            for (int i = 0; i < DPT; i += 4) {
                if (FULL || d0 + i < dim) {
                    const float4 gg = g4[i >> 2], kk = k4[i >> 2];
                    const float ga[4] = {gg.x, gg.y, gg.z, gg.w}, ka[4] = {kk.x, kk.y, kk.z, kk.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        if (FULL || d0 + i + e < dim) {
                            s[i + e] *= ga[e];
                            if (e & 1) dot1 = fmaf(s[i + e], ka[e], dot1);
                            else dot0 = fmaf(s[i + e], ka[e], dot0);
                        }
                }
            }
            float dot = dot0 + dot1;
            dot += __shfl_xor_sync(0xffffffffu, dot, 1);
            dot += __shfl_xor_sync(0xffffffffu, dot, 2);
            const float u = live ? base[o_v + vdim] * (base[o_v + j] - dot) : 0.f;
            float oa = 0.f, ob = 0.f;
#pragma unroll
            for (int i = 0; i < DPT; i += 4) {
                if (FULL || d0 + i < dim) {
                    const float4 kk = k4[i >> 2], qq = q4[i >> 2];
                    const float ka[4] = {kk.x, kk.y, kk.z, kk.w}, qa[4] = {qq.x, qq.y, qq.z, qq.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        if (FULL || d0 + i + e < dim) {
                            s[i + e] = fmaf(ka[e], u, s[i + e]);
                            if (e & 1) ob = fmaf(s[i + e], qa[e], ob);
                            else oa = fmaf(s[i + e], qa[e], oa);
                        }
                }
            }
            float o = oa + ob;
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (live && part == 0) a.o[(size_t)(row0 + c0 + tt) * ((size_t)a.heads * vdim) + (size_t)h * vdim + j] = o;
        }
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < DPT; ++i)
            if (d0 + i < dim) S[(size_t)(d0 + i) * vdim + j] = s[i];
    }
}

// o[t, h, :] <- o / sqrt(mean(o^2) + eps) * w * act(gate[t, h, :]), one warp per (token, head); act = sigmoid or silu;
// gate rows have stride ldg
__global__ void __launch_bounds__(128)
delta_out_kernel(float* __restrict__ o, const float* __restrict__ gate, const float* __restrict__ w, int vdim, float eps,
                 int n_pairs, int heads, int ldg, int gate_act) {
    const int pair = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (pair >= n_pairs) return;
    float* p = o + (size_t)pair * vdim;
    const float* g = gate + (size_t)(pair / heads) * ldg + (size_t)(pair % heads) * vdim;
    float ss = 0.f;
    for (int c = lane; c < vdim; c += 32) ss += p[c] * p[c];
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / (float)vdim + eps);
    for (int c = lane; c < vdim; c += 32) p[c] = p[c] * r * w[c] * sigmoid_exact(g[c]) * (gate_act == 1 ? g[c] : 1.f);
}

int launch_delta(const DeltaArgs& a, const float* gate, const float* out_norm, float eps, int T, int n_req,
                 cudaStream_t stream, int ldg, int gate_act) {
    const int ch = 2 * a.kvh * a.dim + a.heads * a.vdim;
    FT_REQUIRE(a.taps >= 1 && a.taps <= 17, "channel delta: %d convolution taps are beyond 17", a.taps);
    FT_REQUIRE(a.dim <= 256 && a.vdim <= 256, "channel delta: head sizes %d / %d are beyond 256", a.dim, a.vdim);
    FT_REQUIRE((size_t)ch * 4 <= 200 * 1024, "channel delta: %d channels do not fit in shared memory", ch);
    static PerDeviceFlag attr;
    if (!attr.done()) {
        FT_CHECK_CUDA(cudaFuncSetAttribute(delta_prep_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        attr.mark();
    }
    delta_prep_kernel<<<T, 256, (size_t)ch * 4, stream>>>(a);
    FT_CHECK_CUDA(cudaGetLastError());
    if (a.taps > 1) {
        delta_tail_kernel<<<dim3((ch + 127) / 128, n_req), 128, 0, stream>>>(a, n_req);
        FT_CHECK_CUDA(cudaGetLastError());
    }
    const int threads = (4 * std::min(a.vdim, DCOLS) + 31) / 32 * 32;      // four lanes per state column, whole warps
    const int dpt = a.dim <= 32 ? 8 : a.dim <= 64 ? 16 : a.dim <= 128 ? 32 : 64;
    const size_t smem = (size_t)2 * DCHUNK * delta_token_floats(dpt, a.vdim) * 4;
    const dim3 grid(n_req, a.heads, (a.vdim + DCOLS - 1) / DCOLS);
#define FT_DELTA_ONE(DPT_, FULL_)                                                                           \
    do {                                                                                                    \
        if (smem > 48 * 1024)                                                                               \
            FT_CHECK_CUDA(cudaFuncSetAttribute(delta_rule_kernel<DPT_, 4 * DCOLS, FULL_>,                   \
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));    \
        delta_rule_kernel<DPT_, 4 * DCOLS, FULL_><<<grid, threads, smem, stream>>>(a);                      \
    } while (0)
#define FT_DELTA(DPT_)                                  \
    do {                                                \
        if (a.dim == 4 * DPT_) FT_DELTA_ONE(DPT_, true); \
        else FT_DELTA_ONE(DPT_, false);                 \
    } while (0)
    if (a.dim <= 32) FT_DELTA(8);
    else if (a.dim <= 64) FT_DELTA(16);
    else if (a.dim <= 128) FT_DELTA(32);
    else FT_DELTA(64);
#undef FT_DELTA
#undef FT_DELTA_ONE
    FT_CHECK_CUDA(cudaGetLastError());
    const int n_pairs = T * a.heads;
    delta_out_kernel<<<(n_pairs + 3) / 4, 128, 0, stream>>>(a.o, gate, out_norm, a.vdim, eps, n_pairs, a.heads,
                                                            ldg > 0 ? ldg : a.heads * a.vdim, gate_act);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

// ------------------------------------------------------------------ router
// One warp per token: z = logits (+ bias); s = softmax(z) over all E experts (or sigmoid(z) of each); a group's score is its largest s; only
// experts of the `keep` best groups can be chosen; the `top` largest s among them, lowest index first on a tie; weights = s
// as it is, or (normalise) divided by the sum of the chosen ones (+ 1e-20); then times `scale`.
__global__ void __launch_bounds__(128)
route_kernel(const float* __restrict__ proj, int ldp, int o_router, int E, int top, int groups, int keep, int* __restrict__ ids,
             float* __restrict__ wts, int T, int sigmoid_scores, int normalise, float scale, const float* __restrict__ bias) {
    extern __shared__ float sh[];
    const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * (blockDim.x >> 5) + wid;
    if (t >= T) return;
    float* s = sh + (size_t)wid * (E + groups);     // scores, then group scores; a taken entry is set to -1
    float* gs = s + E;
    const float* z = proj + (size_t)t * ldp + o_router;
    if (sigmoid_scores) {
        for (int e = lane; e < E; e += 32) s[e] = sigmoid_exact(z[e] + (bias ? bias[e] : 0.f));
    } else {
        float m = -INFINITY;
        for (int e = lane; e < E; e += 32) {
            s[e] = z[e] + (bias ? bias[e] : 0.f);
            m = fmaxf(m, s[e]);
        }
        m = warp_max(m);
        float sum = 0.f;
        for (int e = lane; e < E; e += 32) { const float v = expf(s[e] - m); s[e] = v; sum += v; }
        sum = warp_sum(sum);
        __syncwarp();
        for (int e = lane; e < E; e += 32) s[e] = s[e] / sum;
    }
    __syncwarp();
    const int per = E / groups;
    for (int g = lane; g < groups; g += 32) {
        float b = -1.f;
        for (int i = 0; i < per; ++i) b = fmaxf(b, s[g * per + i]);
        gs[g] = b;
    }
    __syncwarp();
    // drop the groups that are not among the best `keep`: groups - keep rounds of "remove the smallest" would favour the
    // wrong side of ties, so pick the best `keep` and mark them by negating (score + 2)
    for (int r = 0; r < keep; ++r) {
        float bv = -1.f; int bi = 0x7fffffff;
        for (int g = lane; g < groups; g += 32) if (gs[g] >= 0.f && (gs[g] > bv)) { bv = gs[g]; bi = g; }
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
        }
        if (lane == 0 && bi < groups) gs[bi] = -(bv + 2.f);
        __syncwarp();
    }
    for (int r = 0; r < top; ++r) {
        float bv = -1.f; int bi = 0x7fffffff;
        for (int e = lane; e < E; e += 32)
            if (gs[e / per] < -1.f && s[e] >= 0.f && s[e] > bv) { bv = s[e]; bi = e; }
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
        }
        if (lane == 0) {
            const int e = bi < E ? bi : 0;
            ids[(size_t)t * top + r] = e;
            wts[(size_t)t * top + r] = bi < E ? bv : 0.f;
            if (bi < E) s[bi] = -1.f;
        }
        __syncwarp();
    }
    if (lane == 0 && (normalise || scale != 1.f)) {
        float* w = wts + (size_t)t * top;
        float total = 0.f;
        for (int r = 0; r < top; ++r) total += w[r];
        for (int r = 0; r < top; ++r) w[r] = (normalise ? w[r] / (total + 1e-20f) : w[r]) * scale;
    }
}

// Counting sort of the T * top (token, choice) pairs by expert, one CTA: seg[e] .. seg[e+1] are the sorted places of
// expert e, slot_token[place] the token whose row the expert reads, slot_pos[pair] the place of a pair.  Within an expert the
// order is (token, choice) order, so the layout is the same from run to run.
__global__ void __launch_bounds__(1024)
route_sort_kernel(const int* __restrict__ ids, int n_pairs, int top, int E, int* __restrict__ seg, int* __restrict__ slot_token,
                  int* __restrict__ slot_pos) {
    extern __shared__ int shi[];
    int* cnt = shi;                    // [E + 1]
    for (int e = threadIdx.x; e <= E; e += blockDim.x) cnt[e] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) atomicAdd(&cnt[ids[i] + 1], 1);
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int e = 0; e < E; ++e) cnt[e + 1] += cnt[e];
        for (int e = 0; e <= E; ++e) seg[e] = cnt[e];
    }
    __syncthreads();
    // stable placement: a warp per expert walks the pairs in order (ballot + prefix count)
    const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    for (int e = wid; e < E; e += nw) {
        int base = cnt[e];
        for (int i0 = 0; i0 < n_pairs; i0 += 32) {
            const int i = i0 + lane;
            const bool mine = i < n_pairs && ids[i] == e;
            const unsigned b = __ballot_sync(0xffffffffu, mine);
            if (mine) {
                const int place = base + __popc(b & ((1u << lane) - 1u));
                slot_token[place] = i / top;
                slot_pos[i] = place;
            }
            base += __popc(b);
        }
    }
}

int launch_route(const float* proj, int ldp, int o_router, int E, int top, int groups, int keep, int* ids, float* wts,
                 int* seg, int* slot_token, int* slot_pos, int T, cudaStream_t stream, int route_kind, int normalise,
                 float scale, const float* bias) {
    FT_REQUIRE(groups >= 1 && E % groups == 0 && keep >= 1 && keep <= groups && top >= 1 && top <= (E / groups) * keep,
               "router: %d experts, %d groups, keep %d, top %d do not fit together", E, groups, keep, top);
    const size_t smem = (size_t)4 * (E + groups) * 4;
    FT_REQUIRE(smem <= 48 * 1024 && (size_t)(E + 1) * 4 <= 48 * 1024, "router: %d experts are too many", E);
    route_kernel<<<(T + 3) / 4, 128, smem, stream>>>(proj, ldp, o_router, E, top, groups, keep, ids, wts, T,
                                                     route_kind == FT_ROUTE_SIGMOID, normalise, scale > 0.f ? scale : 1.f, bias);
    FT_CHECK_CUDA(cudaGetLastError());
    route_sort_kernel<<<1, 1024, (size_t)(E + 1) * 4, stream>>>(ids, T * top, top, E, seg, slot_token, slot_pos);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace ft
