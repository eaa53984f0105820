// Retention: linear attention with one constant decay per head, S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, queries and keys
// rotated, every head's result divided by its own root mean square and gated.  Two forms besides the token-by-token rule of
// branches.cu:
//
//   one token per request   retention_step_kernel, one CTA per (request, head), all fp32: rotation, state update, read-out, norm and
//                           gate in one pass over the state (16-byte loads and stores, several rows in flight per thread)
//   prompt portions         in runs of up to 128 tokens, all of them at once, on tcgen05.  With d the decay and n the run's length:
//     retention_pack        rotated q, k (times k_scale) and v as bf16 rows of whole 64-column blocks
//     retention_gain        what a run adds to the state, U = sum_j d^(n-1-j) k_j v_j^T: the decayed keys are fp32 numbers split
//                           into bf16 hi + lo planes (two products into one fp32 accumulator)
//     retention_carry       S <- d^n S + U over the runs of a request in order, fp32; leaves with every run the state it starts from
//     retention_runs        o_i = sum_{j<=i} d^(i-j) (q_i . k_j) v_j + d^(i+1) S^T q_i: scores in fp32, times their decay, as hi + lo
//                           planes in tensor memory; the state as hi + lo planes in shared memory; then norm, gate, bf16 planes
//   Only the projections themselves (q, k, v) are rounded to bf16; decays, scores and the state keep about 16 bits or fp32.
//
// Every wait has a limit; a CTA whose wait runs out marks `err` and returns.
#include "common.cuh"
#include "ft_internal.h"
#include "rows.cuh"

#include <algorithm>

namespace ft {
namespace {

constexpr int RT_RUN = 128, RT_THREADS = 256, RT_SPIN = 1 << 20;
constexpr int RT_BLK = RT_RUN * 128;                    // bytes of one [128 tokens][64 columns] block

__device__ __forceinline__ float gate_value(float g, int act) {
    const float s = sigmoid_quick(g);
    return act ? g * s : s;
}
__device__ __forceinline__ bool rt_wait(uint64_t* bar, uint32_t parity) {
    for (int i = 0; i < RT_SPIN; ++i)
        if (mbar_try_wait(bar, parity)) return true;
    return false;
}
// coordinate c of a rotated head row x: pairs (2i, 2i + 1) or (i, i + dims / 2), cosine and sine of pair i at trig[i], trig[half + i]
__device__ __forceinline__ float turned(const float* __restrict__ x, int c, int dims, int half_layout, const float* trig) {
    if (c >= dims) return x[c];
    const int half = dims >> 1;
    const bool second = half_layout ? c >= half : (c & 1);
    const int i = half_layout ? (second ? c - half : c) : c >> 1;
    const int oc = half_layout ? (second ? c - half : c + half) : (second ? c - 1 : c + 1);
    const float cs = trig[i], sn = trig[half + i];
    return second ? x[c] * cs + x[oc] * sn : x[c] * cs - x[oc] * sn;
}

// ------------------------------------------------------------------ one token per request
template <int CV>
__global__ void __launch_bounds__(RT_THREADS) retention_step_kernel(RetentionArgs a) {
    extern __shared__ __align__(16) float rs_smem[];
    const int D = a.dim, V = a.vdim, h = blockIdx.x, r = blockIdx.y, t = a.req_start[r], tid = threadIdx.x;
    float* sq = rs_smem;                                 // [D]
    float* sk = sq + D;                                  // [D]
    float* trig = sk + D;                                // [rot_dims]
    float* red = trig + a.rot_dims;                      // [33]
    float* sv = rs_smem + ((2 * D + a.rot_dims + 33 + 3) & ~3);      // [V]
    float* so = sv + ((V + 3) & ~3);                     // [V]
    float* part = so + ((V + 3) & ~3);                   // [threads][CV]
    const float* pr = a.proj + (size_t)t * a.ldp;
    const float pos = (float)a.positions[t];
    for (int i = tid; i < a.rot_dims / 2; i += RT_THREADS) sincosf(pos * a.rot_freq[i], &trig[a.rot_dims / 2 + i], &trig[i]);
    for (int c = tid; c < V; c += RT_THREADS) sv[c] = pr[a.o_v + h * V + c];
    __syncthreads();
    for (int c = tid; c < D; c += RT_THREADS) {
        sq[c] = turned(pr + a.o_q + h * D, c, a.rot_dims, a.rot_half, trig);
        sk[c] = turned(pr + a.o_k + h * D, c, a.rot_dims, a.rot_half, trig) * a.k_scale;
    }
    __syncthreads();
    float* S = a.state + (size_t)a.req_slot[r] * a.slot_stride + a.s_off + (size_t)h * D * V;
    const bool old = a.req_pos0[r] > 0;
    const float dec = a.decay[h];
    const int units = V / CV, NC = min(units, RT_THREADS), RG = RT_THREADS / NC;      // column units side by side, row groups
    const int u0 = tid % NC, rg = tid / NC;
    float ss = 0.f;
    for (int ub = 0; ub < units; ub += NC) {
        const int u = ub + u0;
        float o[CV];
#pragma unroll
        for (int i = 0; i < CV; ++i) o[i] = 0.f;
        if (u < units && rg < RG) {
            float v[CV];
#pragma unroll
            for (int i = 0; i < CV; ++i) v[i] = sv[u * CV + i];
            constexpr int NB = 8;                        // state rows on their way at a time
            for (int d0 = rg; d0 < D; d0 += RG * NB) {
                float s[NB][CV];
#pragma unroll
                for (int b = 0; b < NB; ++b) {
                    const int d = d0 + b * RG;
#pragma unroll
                    for (int i = 0; i < CV; ++i) s[b][i] = 0.f;
                    if (old && d < D) ld_cols<CV>(s[b], S + (size_t)d * V + u * CV);
                }
#pragma unroll
                for (int b = 0; b < NB; ++b) {
                    const int d = d0 + b * RG;
                    if (d >= D) break;
                    const float k = sk[d], q = sq[d];
#pragma unroll
                    for (int i = 0; i < CV; ++i) {
                        s[b][i] = fmaf(dec, s[b][i], k * v[i]);
                        o[i] = fmaf(s[b][i], q, o[i]);
                    }
                    st_cols<CV>(S + (size_t)d * V + u * CV, s[b]);
                }
            }
        }
        __syncthreads();
        st_cols<CV>(part + tid * CV, o);
        __syncthreads();
        for (int c = tid; c < NC * CV; c += RT_THREADS) {
            const int col = ub * CV + c;
            if (col >= V) continue;
            float x = 0.f;
            for (int g = 0; g < RG; ++g) x += part[(g * NC + c / CV) * CV + c % CV];
            so[col] = x;
            ss = fmaf(x, x, ss);
        }
    }
    const float rr = 1.f / sqrtf(cta_total(ss, red) / (float)V + a.eps);
    for (int c = tid; c < V; c += RT_THREADS) {
        const float v = so[c] * rr * gate_value(pr[a.o_g + h * V + c], a.gate_act);
        const size_t at = ((size_t)t * a.heads + h) * V + c;
        if (a.out_hi) {
            const __nv_bfloat16 hi = __float2bfloat16_rn(v);
            ((__nv_bfloat16*)a.out_hi)[at] = hi;
            ((__nv_bfloat16*)a.out_lo)[at] = __float2bfloat16_rn(v - __bfloat162float(hi));
        } else {
            a.out[at] = v;
        }
    }
}

// ------------------------------------------------------------------ portions: bf16 rows
// q16, k16 [row][heads][Dp], v16 [row][heads][Vp] of the step's rows from `row0` on (row index counted from there)
__global__ void __launch_bounds__(256) retention_pack_kernel(RetentionArgs a, int row0, int Dp, int Vp) {
    extern __shared__ float trig[];
    const int t = row0 + blockIdx.x, H = a.heads, D = a.dim, V = a.vdim, half = a.rot_dims >> 1;
    const float* pr = a.proj + (size_t)t * a.ldp;
    const float pos = (float)a.positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * a.rot_freq[i], &trig[half + i], &trig[i]);
    __syncthreads();
    const int dch = Dp / 8, vch = Vp / 8, per = 2 * dch + vch;
    // whole 8-column pieces whose partners are a whole piece too
    const bool wide = (D & 7) == 0 && (a.rot_dims == 0 || (a.rot_half && (half & 7) == 0)) && (a.ldp & 3) == 0 && ((a.o_q | a.o_k) & 3) == 0;
    const bool vwide = (V & 7) == 0 && (a.ldp & 3) == 0 && (a.o_v & 3) == 0;
    for (int idx = threadIdx.x; idx < H * per; idx += blockDim.x) {
        const int h = idx / per, p = idx % per;
        const int kind = p < dch ? 0 : p < 2 * dch ? 1 : 2, ch = kind == 0 ? p : kind == 1 ? p - dch : p - 2 * dch, c0 = ch * 8;
        float x[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] = 0.f;
        __nv_bfloat16* dst;
        if (kind == 2) {
            const float* src = pr + a.o_v + h * V;
            if (vwide) {
                if (c0 < V) {
                    const float4 u = *reinterpret_cast<const float4*>(src + c0), v = *reinterpret_cast<const float4*>(src + c0 + 4);
                    x[0] = u.x; x[1] = u.y; x[2] = u.z; x[3] = u.w; x[4] = v.x; x[5] = v.y; x[6] = v.z; x[7] = v.w;
                }
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) if (c0 + i < V) x[i] = src[c0 + i];
            }
            dst = (__nv_bfloat16*)a.v16 + ((size_t)blockIdx.x * H + h) * Vp + c0;
        } else {
            const float* src = pr + (kind == 0 ? a.o_q : a.o_k) + h * D;
            const float sc = kind == 1 ? a.k_scale : 1.f;
            if (wide) {
                if (c0 < D) {
                    const float4 u = *reinterpret_cast<const float4*>(src + c0), v = *reinterpret_cast<const float4*>(src + c0 + 4);
                    x[0] = u.x; x[1] = u.y; x[2] = u.z; x[3] = u.w; x[4] = v.x; x[5] = v.y; x[6] = v.z; x[7] = v.w;
                    if (c0 < a.rot_dims) {
                        const bool second = c0 >= half;
                        const int i0 = second ? c0 - half : c0, oc = second ? c0 - half : c0 + half;
                        const float4 p0 = *reinterpret_cast<const float4*>(src + oc), p1 = *reinterpret_cast<const float4*>(src + oc + 4);
                        const float y[8] = {p0.x, p0.y, p0.z, p0.w, p1.x, p1.y, p1.z, p1.w};
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            const float cs = trig[i0 + i], sn = trig[half + i0 + i];
                            x[i] = second ? x[i] * cs + y[i] * sn : x[i] * cs - y[i] * sn;
                        }
                    }
                }
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) if (c0 + i < D) x[i] = turned(src, c0 + i, a.rot_dims, a.rot_half, trig);
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) x[i] *= sc;
            dst = (__nv_bfloat16*)(kind == 0 ? a.q16 : a.k16) + ((size_t)blockIdx.x * H + h) * Dp + c0;
        }
        *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]), pack_bf16(x[4], x[5]), pack_bf16(x[6], x[7]));
    }
}

// A run of up to 128 tokens: which portion, its first row (from the pack's row 0), its length, its place in the state work buffer.
struct Run { int portion, row, n, slot, q0; };
__device__ __forceinline__ bool find_run(const WindowTiles& tm, int tile, Run& r) {
    r.portion = tm.tile_req[tile];
    r.q0 = tm.tile_q0[tile];
    if (r.q0 % RT_RUN != 0) return false;               // a run of two query tiles belongs to the first of them
    const int start = tm.req_q_start[r.portion];
    r.row = start - tm.req_q_start[0] + r.q0;
    r.n = min(RT_RUN, tm.req_q_start[r.portion + 1] - start - r.q0);
    // tiles of a portion are consecutive, so its first one is tile - q0 / 64; portions round up to whole runs
    r.slot = (tile - r.q0 / kKvTile + r.portion) / 2 + r.q0 / RT_RUN;
    return true;
}

// rows [n_rows] of a bf16 array (row stride ld elements, `blocks` 64-column blocks) -> swizzled blocks of [128 rows][64 columns], by
// asynchronous copies (rows beyond n_rows are filled with zeros); rt_landed() waits for them
__device__ __forceinline__ void rt_landed() { asm volatile("cp.async.wait_all;" ::: "memory"); }
__device__ __forceinline__ void stage_rows(uint8_t* dst, const __nv_bfloat16* src, size_t ld, int blocks, int n_rows) {
    const int ch = threadIdx.x & 7, r0 = threadIdx.x >> 3;
    const uint32_t base = smem_u32(dst);
    for (int b = 0; b < blocks; ++b)
#pragma unroll
        for (int r = r0; r < RT_RUN; r += RT_THREADS / 8) {
            const bool in = r < n_rows;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(base + b * RT_BLK + r * 128 + ((ch ^ (r & 7)) << 4)),
                         "l"(src + (in ? (size_t)r * ld : 0) + b * 64 + ch * 8), "r"(in ? 16 : 0)
                         : "memory");
        }
}
// eight fp32 numbers as bf16 hi and lo pieces
__device__ __forceinline__ void split8(const float (&x)[8], uint4& hi, uint4& lo) {
    uint32_t h[4], l[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        h[e] = pack_bf16(x[2 * e], x[2 * e + 1]);
        l[e] = pack_bf16(x[2 * e] - bf16_lo(h[e]), x[2 * e + 1] - bf16_hi(h[e]));
    }
    hi = make_uint4(h[0], h[1], h[2], h[3]);
    lo = make_uint4(l[0], l[1], l[2], l[3]);
}

// 128 rows x nv columns of TMEM -> tile (row stride ld floats): warps w and w + 4 share the lanes of a quarter
__device__ __forceinline__ void tile_out(float* tile, int ld, uint32_t tmem, int nv, int warp, int lane) {
    const int row = (warp & 3) * 32 + lane;
    for (int c = (warp >> 2) * 16; c < nv; c += 32) {
        float v[16];
        tmem_ld16(tmem + ((uint32_t)((warp & 3) * 32) << 16) + c, v);
#pragma unroll
        for (int i = 0; i < 16; i += 4) *reinterpret_cast<float4*>(tile + row * ld + c + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
        __syncwarp();
    }
}

// ------------------------------------------------------------------ what a run adds to the state
// D[d][v] (TMEM, M = 128 key channels, N = up to 128 value columns) = Kd^T V over the run's tokens; both operands MN-major.
__global__ void __launch_bounds__(RT_THREADS) retention_gain_kernel(RetentionArgs a, WindowTiles tm, int Dp, int Vp, int* err) {
    extern __shared__ uint8_t rg_raw[];
    __shared__ float pw[RT_RUN];
    __shared__ uint64_t done;
    __shared__ uint32_t tmem_slot;
    Run run;
    if (!find_run(tm, blockIdx.x, run)) return;
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rg_raw) + 1023) & ~uintptr_t(1023));
    uint8_t *k_hi = smem, *k_lo = smem + 2 * RT_BLK, *v_s = smem + 4 * RT_BLK;
    const int h = blockIdx.y, v0 = blockIdx.z * 128, nv = min(128, Vp - v0), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        mbar_init(&done, 1);
        fence_mbar_init();
    }
    if (warp == 0) {
        tmem_alloc(&tmem_slot, 128);
        tmem_relinquish();
    }
    if (tid < RT_RUN) pw[tid] = powf(a.decay[h], (float)tid);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    stage_rows(v_s, (const __nv_bfloat16*)a.v16 + ((size_t)run.row * a.heads + h) * Vp + v0, (size_t)a.heads * Vp, nv / 64, run.n);
    const __nv_bfloat16* ks = (const __nv_bfloat16*)a.k16 + ((size_t)run.row * a.heads + h) * Dp;
    {
        const int ch = tid & 7, r0 = tid >> 3;
        constexpr int NR = RT_RUN / (RT_THREADS / 8);    // rows per thread, all of a block's on their way at once
        for (int b = 0; b < Dp / 64; ++b) {
            uint4 k[NR];
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const int r = r0 + i * (RT_THREADS / 8);
                k[i] = make_uint4(0u, 0u, 0u, 0u);
                if (r < run.n) k[i] = *reinterpret_cast<const uint4*>(ks + (size_t)r * a.heads * Dp + b * 64 + ch * 8);
            }
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const int r = r0 + i * (RT_THREADS / 8);
                const float f = pw[max(run.n - 1 - r, 0)];
                const float x[8] = {bf16_lo(k[i].x) * f, bf16_hi(k[i].x) * f, bf16_lo(k[i].y) * f, bf16_hi(k[i].y) * f,
                                    bf16_lo(k[i].z) * f, bf16_hi(k[i].z) * f, bf16_lo(k[i].w) * f, bf16_hi(k[i].w) * f};
                uint4 hi, lo;
                split8(x, hi, lo);
                const int at = b * RT_BLK + r * 128 + ((ch ^ (r & 7)) << 4);
                *reinterpret_cast<uint4*>(k_hi + at) = hi;
                *reinterpret_cast<uint4*>(k_lo + at) = lo;
            }
        }
    }
    rt_landed();
    fence_proxy_async();
    __syncthreads();
    if (tid == 0) {
        const uint32_t idesc = umma_idesc_bf16(128, nv) | (1u << 15) | (1u << 16);      // A and B MN-major
        const uint64_t hd = umma_desc_mn128(smem_u32(k_hi), RT_BLK), ld = umma_desc_mn128(smem_u32(k_lo), RT_BLK),
                       vd = umma_desc_mn128(smem_u32(v_s), RT_BLK);
        const int steps = (run.n + 15) / 16;
        for (int k = 0; k < steps; ++k) {
            umma_bf16(tmem, hd + k * (2048 >> 4), vd + k * (2048 >> 4), idesc, k > 0);
            umma_bf16(tmem, ld + k * (2048 >> 4), vd + k * (2048 >> 4), idesc, 1);
        }
        umma_commit(&done);
    }
    __syncwarp();
    bool ok = rt_wait(&done, 0);
    tc_fence_after();
    __syncwarp();
    ok = __syncthreads_and(ok);
    if (ok) {
        // through shared memory (the operands have been read), so that a warp writes whole rows
        const int ld = nv + 4;
        float* tile = reinterpret_cast<float*>(smem);
        tile_out(tile, ld, tmem, nv, warp, lane);
        __syncthreads();
        float* dst = a.ws + ((size_t)run.slot * a.heads + h) * a.dim * a.vdim + v0;
        const int cols = min(nv, a.vdim - v0);
        if ((a.vdim & 3) == 0) {
            for (int i = tid; i < a.dim * (cols / 4); i += RT_THREADS) {
                const int d = i / (cols / 4), c = i % (cols / 4) * 4;
                *reinterpret_cast<float4*>(dst + (size_t)d * a.vdim + c) = *reinterpret_cast<const float4*>(tile + d * ld + c);
            }
        } else {
            for (int i = tid; i < a.dim * cols; i += RT_THREADS) dst[(size_t)(i / cols) * a.vdim + i % cols] = tile[i / cols * ld + i % cols];
        }
    } else if (tid == 0 && err) {
        *err = 1;
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        tc_fence_after();
        tmem_dealloc(tmem, 128);
    }
}

// ------------------------------------------------------------------ the state from run to run
// ws of a run: what it adds -> what it starts from.  CV numbers per thread.
template <int CV>
__global__ void __launch_bounds__(256) retention_carry_kernel(RetentionArgs a, WindowTiles tm, int first_req) {
    const int j = blockIdx.z, h = blockIdx.y, e = (blockIdx.x * blockDim.x + threadIdx.x) * CV, DV = a.dim * a.vdim;
    if (e >= DV) return;
    const int len = tm.req_q_start[j + 1] - tm.req_q_start[j], n_runs = (len + RT_RUN - 1) / RT_RUN;
    int tile = 0;                                        // the portion's first query tile
    for (int i = 0; i < j; ++i) tile += (tm.req_q_start[i + 1] - tm.req_q_start[i] + kKvTile - 1) / kKvTile;
    const int slot0 = (tile + j) / 2, r = first_req + j;
    const float d_full = powf(a.decay[h], (float)RT_RUN), d_last = powf(a.decay[h], (float)(len - (n_runs - 1) * RT_RUN));
    float* S = a.state + (size_t)a.req_slot[r] * a.slot_stride + a.s_off + (size_t)h * DV + e;
    float s[CV];
#pragma unroll
    for (int i = 0; i < CV; ++i) s[i] = 0.f;
    if (a.req_pos0[r] > 0) ld_cols<CV>(s, S);
    float* w = a.ws + ((size_t)slot0 * a.heads + h) * DV + e;
    const size_t step = (size_t)a.heads * DV;
    constexpr int NB = 8;                                // runs on their way at a time
    for (int c0 = 0; c0 < n_runs; c0 += NB) {
        float u[NB][CV];
#pragma unroll
        for (int b = 0; b < NB; ++b)
            if (c0 + b < n_runs) ld_cols<CV>(u[b], w + (c0 + b) * step);
#pragma unroll
        for (int b = 0; b < NB; ++b) {
            if (c0 + b >= n_runs) break;
            st_cols<CV>(w + (c0 + b) * step, s);
            const float f = c0 + b + 1 < n_runs ? d_full : d_last;
#pragma unroll
            for (int i = 0; i < CV; ++i) s[i] = fmaf(f, s[i], u[b][i]);
        }
    }
    st_cols<CV>(S, s);
}

// ------------------------------------------------------------------ the results of a run
// Two CTAs per SM.  TMEM: scores 0..127, over them their decayed values as planes (hi 0..63, lo 64..127), over those at last the
// state's part; run's part 128..255.  Shared memory: q | k | v; the state's hi plane takes the place of k once the scores are there,
// its lo plane that of v once the run's part is.
constexpr int RT_COL_S = 0, RT_COL_PH = 0, RT_COL_PL = 64, RT_COL_O1 = 0, RT_COL_O2 = 128;
__global__ void __launch_bounds__(RT_THREADS, 2) retention_runs_kernel(RetentionArgs a, WindowTiles tm, int Dp, int Vp, int raw, int first_req, int* err) {
    extern __shared__ uint8_t rr_raw[];
    __shared__ float pw[RT_RUN + 1];
    __shared__ uint64_t done[3];
    __shared__ uint32_t tmem_slot;
    Run run;
    if (!find_run(tm, blockIdx.x, run)) return;
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rr_raw) + 1023) & ~uintptr_t(1023));
    const int db = Dp / 64, h = blockIdx.y, v0 = blockIdx.z * 128, nv = min(128, Vp - v0), vb = nv / 64, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int sblk = Dp * 128;                           // bytes of one [Dp channels][64 columns] block of the state
    uint8_t *q_s = smem, *k_s = q_s + db * RT_BLK, *v_s = k_s + db * RT_BLK, *s_hi = k_s, *s_lo = v_s;
    const bool carried = a.req_pos0[first_req + run.portion] > 0 || run.q0 > 0;      // otherwise the state it starts from is zero
    if (tid == 0) {
        for (int i = 0; i < 3; ++i) mbar_init(&done[i], 1);
        fence_mbar_init();
    }
    if (warp == 0) {
        tmem_alloc(&tmem_slot, 256);
        tmem_relinquish();
    }
    const size_t hd = (size_t)a.heads * Dp;
    stage_rows(q_s, (const __nv_bfloat16*)a.q16 + ((size_t)run.row * a.heads + h) * Dp, hd, db, run.n);
    stage_rows(k_s, (const __nv_bfloat16*)a.k16 + ((size_t)run.row * a.heads + h) * Dp, hd, db, run.n);
    stage_rows(v_s, (const __nv_bfloat16*)a.v16 + ((size_t)run.row * a.heads + h) * Vp + v0, (size_t)a.heads * Vp, vb, run.n);
    if (tid <= RT_RUN) pw[tid] = powf(a.decay[h], (float)tid);
    rt_landed();
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    if (tid == 0) {
        const uint32_t idesc_qk = umma_idesc_bf16(RT_RUN, RT_RUN);
        for (int b = 0; b < db; ++b) {
            const uint64_t qd = umma_desc_k128(smem_u32(q_s + b * RT_BLK)), kd = umma_desc_k128(smem_u32(k_s + b * RT_BLK));
#pragma unroll
            for (int k = 0; k < 4; ++k) umma_bf16(tmem + RT_COL_S, qd + 2 * k, kd + 2 * k, idesc_qk, (b | k) != 0);
        }
        umma_commit(&done[0]);
    }
    __syncwarp();
    bool ok = rt_wait(&done[0], 0);
    tc_fence_after();
    __syncwarp();
    const int i_row = (warp & 3) * 32 + lane, col_half = warp >> 2;      // TMEM lane == row of the run
    const uint32_t lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    // scores times decay^(i - j), zero above the diagonal
    uint32_t ph[2][16], pl[2][16];
    if (ok) {
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int col = col_half * 64 + x * 32;
            uint32_t s[32];
            tmem_ld16_nowait(lanes + RT_COL_S + col, s);
            tmem_ld16_nowait(lanes + RT_COL_S + col + 16, s + 16);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 16; ++e) {
                const int j = col + 2 * e;
                const float u = j <= i_row ? __uint_as_float(s[2 * e]) * pw[i_row - j] : 0.f;
                const float v = j + 1 <= i_row ? __uint_as_float(s[2 * e + 1]) * pw[i_row - j - 1] : 0.f;
                ph[x][e] = pack_bf16(u, v);
                pl[x][e] = pack_bf16(u - bf16_lo(ph[x][e]), v - bf16_hi(ph[x][e]));
            }
        }
    }
    tc_fence_before();
    ok = __syncthreads_and(ok);                          // every score has been read
    tc_fence_after();
    if (ok) {
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            tmem_st16(lanes + RT_COL_PH + col_half * 32 + x * 16, ph[x]);
            tmem_st16(lanes + RT_COL_PL + col_half * 32 + x * 16, pl[x]);
        }
        tmem_st_wait();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (ok && tid == 0) {
        const uint32_t idesc_pv = umma_idesc_bf16(RT_RUN, nv) | (1u << 16);      // B MN-major
        const uint64_t vd = umma_desc_mn128(smem_u32(v_s), RT_BLK);
        const int steps = (run.n + 15) / 16;
        for (int k = 0; k < steps; ++k) {
            umma_f16_ts(tmem + RT_COL_O2, tmem + RT_COL_PH + 8 * k, vd + k * (2048 >> 4), idesc_pv, k > 0);
            umma_f16_ts(tmem + RT_COL_O2, tmem + RT_COL_PL + 8 * k, vd + k * (2048 >> 4), idesc_pv, 1);
        }
        umma_commit(&done[1]);
    }
    __syncwarp();
    // the state meanwhile: hi plane to its place, lo plane in registers until the values have been read
    constexpr int ND = 4, ST = RT_THREADS / 8;           // channels per thread and block, their stride
    const int ch = tid & 7, d0 = tid >> 3;
    uint4 lo[2][ND];
    if (carried) {
        const float* ws = a.ws + ((size_t)run.slot * a.heads + h) * a.dim * a.vdim;
        const bool v4 = (a.vdim & 3) == 0;
#pragma unroll
        for (int b = 0; b < 2; ++b) {
            if (b >= vb) break;
            const int c = v0 + b * 64 + ch * 8;
            float x[ND][8];
#pragma unroll
            for (int i = 0; i < ND; ++i) {
                const int d = d0 + i * ST;
#pragma unroll
                for (int e = 0; e < 8; ++e) x[i][e] = 0.f;
                if (d < a.dim) {
                    const float* src = ws + (size_t)d * a.vdim + c;
                    if (v4) {
                        if (c < a.vdim) { const float4 t = *reinterpret_cast<const float4*>(src); x[i][0] = t.x; x[i][1] = t.y; x[i][2] = t.z; x[i][3] = t.w; }
                        if (c + 4 < a.vdim) { const float4 t = *reinterpret_cast<const float4*>(src + 4); x[i][4] = t.x; x[i][5] = t.y; x[i][6] = t.z; x[i][7] = t.w; }
                    } else {
#pragma unroll
                        for (int e = 0; e < 8; ++e) if (c + e < a.vdim) x[i][e] = src[e];
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < ND; ++i) {
                const int d = d0 + i * ST;
                uint4 hi;
                split8(x[i], hi, lo[b][i]);
                if (d < Dp) *reinterpret_cast<uint4*>(s_hi + b * sblk + d * 128 + ((ch ^ (d & 7)) << 4)) = hi;
            }
        }
    }
    if (ok) ok = rt_wait(&done[1], 0);
    tc_fence_after();
    __syncwarp();
    if (carried) {                                       // the same for the whole CTA
        if (ok) {
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                if (b >= vb) break;
#pragma unroll
                for (int i = 0; i < ND; ++i) {
                    const int d = d0 + i * ST;
                    if (d < Dp) *reinterpret_cast<uint4*>(s_lo + b * sblk + d * 128 + ((ch ^ (d & 7)) << 4)) = lo[b][i];
                }
            }
        }
        fence_proxy_async();
        tc_fence_before();
        ok = __syncthreads_and(ok);
        tc_fence_after();
        if (ok && tid == 0) {
            const uint32_t idesc_qs = umma_idesc_bf16(RT_RUN, nv) | (1u << 16);
            const uint64_t sh = umma_desc_mn128(smem_u32(s_hi), sblk), sl = umma_desc_mn128(smem_u32(s_lo), sblk);
            for (int b = 0; b < db; ++b) {
                const uint64_t qd = umma_desc_k128(smem_u32(q_s + b * RT_BLK));
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const uint64_t off = (uint64_t)((b * 4 + k) * 2048) >> 4;
                    umma_bf16(tmem + RT_COL_O1, qd + 2 * k, sh + off, idesc_qs, (b | k) != 0);
                    umma_bf16(tmem + RT_COL_O1, qd + 2 * k, sl + off, idesc_qs, 1);
                }
            }
            umma_commit(&done[2]);
        }
        __syncwarp();
        if (ok) ok = rt_wait(&done[2], 0);
        tc_fence_after();
        __syncwarp();
    }
    ok = __syncthreads_and(ok);
    if (ok) {
        // through shared memory (all operands have been read): then a warp per row
        const int ld = nv + 4;
        float* tile = reinterpret_cast<float*>(smem);
        const float after = pw[min(i_row + 1, RT_RUN)];
        for (int c = col_half * 16; c < nv; c += 32) {
            float o[16], x[16];
            tmem_ld16(lanes + RT_COL_O2 + c, o);
            if (carried) {
                tmem_ld16(lanes + RT_COL_O1 + c, x);
#pragma unroll
                for (int i = 0; i < 16; ++i) o[i] = fmaf(after, x[i], o[i]);
            }
#pragma unroll
            for (int i = 0; i < 16; i += 4) *reinterpret_cast<float4*>(tile + i_row * ld + c + i) = make_float4(o[i], o[i + 1], o[i + 2], o[i + 3]);
            __syncwarp();
        }
        __syncthreads();
        __nv_bfloat16 *oh = (__nv_bfloat16*)a.out_hi, *ol = (__nv_bfloat16*)a.out_lo;
        const bool v4 = (a.vdim & 3) == 0 && (a.ldp & 3) == 0 && (a.o_g & 3) == 0;
        const int row0 = tm.req_q_start[0] + run.row, cols = min(nv, a.vdim - v0);
        constexpr int NR = 4;                            // rows of a warp on their way at a time
        for (int r0 = warp; r0 < run.n; r0 += NR * (RT_THREADS / 32)) {
            if (v4) {
                float4 g[NR];
                const int c = lane * 4;
#pragma unroll
                for (int i = 0; i < NR; ++i) {
                    const int r = r0 + i * (RT_THREADS / 32);
                    g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (!raw && r < run.n && c < cols) g[i] = *reinterpret_cast<const float4*>(a.proj + (size_t)(row0 + r) * a.ldp + a.o_g + h * a.vdim + c);
                }
#pragma unroll
                for (int i = 0; i < NR; ++i) {
                    const int r = r0 + i * (RT_THREADS / 32);
                    if (r >= run.n) break;
                    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (c < cols) v = *reinterpret_cast<const float4*>(tile + r * ld + c);
                    const size_t at = ((size_t)(row0 + r) * a.heads + h) * a.vdim + v0 + c;
                    if (!raw) {
                        const float rr = 1.f / sqrtf(warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w) / (float)a.vdim + a.eps);
                        v.x *= rr * gate_value(g[i].x, a.gate_act); v.y *= rr * gate_value(g[i].y, a.gate_act);
                        v.z *= rr * gate_value(g[i].z, a.gate_act); v.w *= rr * gate_value(g[i].w, a.gate_act);
                    }
                    if (c >= cols) continue;
                    if (oh && !raw) {
                        const uint32_t h0 = pack_bf16(v.x, v.y), h1 = pack_bf16(v.z, v.w);
                        *reinterpret_cast<uint2*>(oh + at) = make_uint2(h0, h1);
                        *reinterpret_cast<uint2*>(ol + at) = make_uint2(pack_bf16(v.x - bf16_lo(h0), v.y - bf16_hi(h0)),
                                                                        pack_bf16(v.z - bf16_lo(h1), v.w - bf16_hi(h1)));
                    } else {
                        *reinterpret_cast<float4*>(a.out + at) = v;
                    }
                }
            } else {
                for (int i = 0; i < NR; ++i) {
                    const int r = r0 + i * (RT_THREADS / 32);
                    if (r >= run.n) break;
                    float ss = 0.f;
                    for (int c = lane; c < cols; c += 32) ss = fmaf(tile[r * ld + c], tile[r * ld + c], ss);
                    const float rr = raw ? 1.f : 1.f / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
                    const float* gate = a.proj + (size_t)(row0 + r) * a.ldp + a.o_g + h * a.vdim;
                    for (int c = lane; c < cols; c += 32) {
                        float v = tile[r * ld + c];
                        if (!raw) v *= rr * gate_value(gate[c], a.gate_act);
                        const size_t at = ((size_t)(row0 + r) * a.heads + h) * a.vdim + v0 + c;
                        if (oh && !raw) {
                            const __nv_bfloat16 b = __float2bfloat16_rn(v);
                            oh[at] = b;
                            ol[at] = __float2bfloat16_rn(v - __bfloat162float(b));
                        } else {
                            a.out[at] = v;
                        }
                    }
                }
            }
        }
    } else if (tid == 0 && err) {
        *err = 1;
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        tc_fence_after();
        tmem_dealloc(tmem, 256);
    }
}

int pad64(int n) { return (n + 63) / 64 * 64; }
size_t runs_smem(int dim, int vdim) {
    const int Dp = pad64(dim), nv = std::min(pad64(vdim), 128);
    return 1024 + std::max((size_t)(2 * (Dp / 64) + nv / 64) * RT_BLK, (size_t)RT_RUN * (nv + 4) * 4);
}
constexpr size_t RT_GAIN_SMEM = 1024 + 6 * RT_BLK;

}  // namespace

// state slots of the work buffer for a step of `rows` portion rows in `portions` portions
int retention_ws_runs(int rows, int portions) { return rows / RT_RUN + portions + 1; }
bool retention_tc_ok(int dim, int vdim) { return dim >= 1 && dim <= 128 && vdim >= 1; }
bool retention_one_pass(int vdim) { return vdim <= 128; }
int retention_padded(int n) { return pad64(n); }

int launch_retention_step(const RetentionArgs& a, int n_req, cudaStream_t stream) {
    if (n_req <= 0) return 0;
    FT_REQUIRE(a.proj && a.state && a.decay && (a.rot_dims == 0 || a.rot_freq) && (a.out || a.out_hi) && n_req <= 65535, "retention step: missing operands");
    const bool v4 = a.vdim % 4 == 0 && a.slot_stride % 4 == 0 && a.s_off % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    const int cv = v4 ? 4 : 1;
    const size_t smem = (size_t)(((2 * a.dim + a.rot_dims + 33 + 3) & ~3) + 2 * ((a.vdim + 3) & ~3) + RT_THREADS * cv) * 4;
    FT_REQUIRE(smem <= 48 * 1024, "retention step: head sizes %d / %d are too large", a.dim, a.vdim);
    const dim3 grid(a.heads, n_req);
    if (v4) retention_step_kernel<4><<<grid, RT_THREADS, smem, stream>>>(a);
    else retention_step_kernel<1><<<grid, RT_THREADS, smem, stream>>>(a);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

int launch_retention_tc(const RetentionArgs& a, const WindowTiles& tm, int first_req, int row0, int rows, int portions, int* err, cudaStream_t stream) {
    FT_REQUIRE(retention_tc_ok(a.dim, a.vdim) && a.q16 && a.k16 && a.v16 && a.ws && portions <= 65535, "retention (tcgen05): sizes %d / %d do not fit", a.dim, a.vdim);
    const int Dp = pad64(a.dim), Vp = pad64(a.vdim), groups = (Vp + 127) / 128;
    static PerDeviceFlag attr;
    if (!attr.done()) {
        FT_CHECK_CUDA(cudaFuncSetAttribute(retention_gain_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)RT_GAIN_SMEM));
        FT_CHECK_CUDA(cudaFuncSetAttribute(retention_runs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024));
        attr.mark();
    }
    retention_pack_kernel<<<rows, 256, (size_t)a.rot_dims * 4, stream>>>(a, row0, Dp, Vp);
    FT_CHECK_CUDA(cudaGetLastError());
    const dim3 grid(tm.n_tiles, a.heads, groups);
    retention_gain_kernel<<<grid, RT_THREADS, RT_GAIN_SMEM, stream>>>(a, tm, Dp, Vp, err);
    FT_CHECK_CUDA(cudaGetLastError());
    const int dv = a.dim * a.vdim;
    const bool v4 = a.vdim % 4 == 0 && a.slot_stride % 4 == 0 && a.s_off % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    if (v4) retention_carry_kernel<4><<<dim3((dv / 4 + 255) / 256, a.heads, portions), 256, 0, stream>>>(a, tm, first_req);
    else retention_carry_kernel<1><<<dim3((dv + 255) / 256, a.heads, portions), 256, 0, stream>>>(a, tm, first_req);
    FT_CHECK_CUDA(cudaGetLastError());
    retention_runs_kernel<<<grid, RT_THREADS, runs_smem(a.dim, a.vdim), stream>>>(a, tm, Dp, Vp, !retention_one_pass(a.vdim), first_req, err);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace ft
