// Softmax attention over the paged bf16 cache (Paged16Args): what fills the cache for window-attention branches, the attention of
// single tokens on mma.sync with the keys cut into shares, and the merge of the shares.
#include "common.cuh"
#include "ft_internal.h"

#include <algorithm>

namespace ft {
namespace {

__device__ __forceinline__ float sigmoid_full(float z) { return 1.f / (1.f + expf(-z)); }

// ------------------------------------------------------------------ queries, keys and values of a step
// One warp per (token, head) over the query heads, then the key heads, then the value heads: bias, norm over the head, gain,
// rotation, and for a query temperature and score scale; bf16, zeros up to whole 64-column blocks.
constexpr int PW_WARPS = 4;
__global__ void __launch_bounds__(PW_WARPS * 32) paged16_write_kernel(WindowArgs a, __nv_bfloat16* __restrict__ q16, __nv_bfloat16* __restrict__ cache,
                                                                      int key_blocks, int v_blocks, int row_floats) {
    extern __shared__ __align__(16) float pw_rows[];
    const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x;
    const int hh = blockIdx.y * PW_WARPS + wid;
    if (hh >= a.H + 2 * a.G) return;
    float* row = pw_rows + (size_t)wid * row_floats;
    const int kind = hh < a.H ? 0 : hh < a.H + a.G ? 1 : 2;               // query, key, value
    const int h = kind == 0 ? hh : (hh - a.H) % a.G, n = kind == 2 ? a.vdim : a.dim;
    const float* src = a.proj + (size_t)t * a.ldp + (kind == 0 ? a.o_q : kind == 1 ? a.o_k : a.o_v) + h * n;
    const float* bias = kind == 0 ? a.q_bias : kind == 1 ? a.k_bias : a.v_bias;
    const float* gain = kind == 0 ? a.q_gain : kind == 1 ? a.k_gain : nullptr;
    const int pos = a.positions[t];
    const int padded = (kind == 2 ? v_blocks : key_blocks) * 64;
    float ss = 0.f;
    for (int c = lane; c < padded; c += 32) {
        float v = c < n ? src[c] : 0.f;
        if (bias && c < n) v += bias[h * n + c];
        row[c] = v;
        ss = fmaf(v, v, ss);
    }
    __syncwarp();
    if (kind < 2) {
        float f = 1.f;
        if (a.qk_norm) f = 1.f / sqrtf(warp_sum(ss) / (float)n + a.eps);
        float late = 1.f;                                                 // after the rotation
        if (kind == 0) {
            late = a.scale;
            if (a.temp_every > 0) late *= fmaf(a.temp_coef, logf((float)((pos + 1) / a.temp_every + 1)), 1.f);
        }
        if (a.rot_dims > 0) {
            for (int c = lane; c < n; c += 32) row[c] *= gain ? f * gain[c] : f;
            __syncwarp();
            const int half = a.rot_dims >> 1;
            for (int i = lane; i < half; i += 32) {
                const int i0 = a.rot_half ? i : 2 * i, i1 = a.rot_half ? i + half : 2 * i + 1;
                float sn, cs;
                sincosf((float)pos * a.rot_freq[i], &sn, &cs);
                sn *= a.rot_mag;
                cs *= a.rot_mag;
                const float u = row[i0], v = row[i1];
                row[i0] = u * cs - v * sn;
                row[i1] = v * cs + u * sn;
            }
            __syncwarp();
            for (int c = lane; c < n; c += 32) row[c] *= late;
        } else {
            for (int c = lane; c < n; c += 32) row[c] *= (gain ? f * gain[c] : f) * late;
        }
        __syncwarp();
    }
    __nv_bfloat16* dst;
    if (kind == 0) {
        dst = q16 + ((size_t)t * a.H + h) * padded;
    } else {
        const int page = a.page_table[(size_t)a.seq_rows[t] * a.max_pages + pos / kKvTile];
        dst = cache + ((size_t)page * a.G + h) * (size_t)(key_blocks + v_blocks) * (kKvTile * 64) + (kind == 2 ? (size_t)key_blocks * (kKvTile * 64) : 0);
    }
    for (int ch = lane; ch < padded / 8; ch += 32) {
        const float4 u = *reinterpret_cast<const float4*>(row + ch * 8), v = *reinterpret_cast<const float4*>(row + ch * 8 + 4);
        const uint4 o = make_uint4(pack_bf16(u.x, u.y), pack_bf16(u.z, u.w), pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
        *reinterpret_cast<uint4*>(dst + (kind == 0 ? ch * 8 : latent_chunk16(pos % kKvTile, ch))) = o;
    }
}

// The same without rotation and bias, rows on 16-byte boundaries: NV float4s of the head per lane stay in registers, NH heads per
// warp have their loads in flight together.
template <int NV, int NH>
__global__ void __launch_bounds__(PW_WARPS * 32) paged16_write_rows_kernel(WindowArgs a, __nv_bfloat16* __restrict__ q16,
                                                                           __nv_bfloat16* __restrict__ cache, int key_blocks, int v_blocks) {
    const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x;
    const int hh0 = (blockIdx.y * PW_WARPS + wid) * NH, n_heads = a.H + 2 * a.G;
    if (hh0 >= n_heads) return;
    const int pos = a.positions[t];
    const int page = a.page_table[(size_t)a.seq_rows[t] * a.max_pages + pos / kKvTile];
    float4 v[NH][NV];
#pragma unroll
    for (int j = 0; j < NH; ++j) {
        const int hh = hh0 + j, kind = hh < a.H ? 0 : hh < a.H + a.G ? 1 : 2, h = kind == 0 ? hh : (hh - a.H) % a.G, n = kind == 2 ? a.vdim : a.dim;
        const float* src = a.proj + (size_t)t * a.ldp + (kind == 0 ? a.o_q : kind == 1 ? a.o_k : a.o_v) + h * n;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (i * 32 + lane) * 4;
            v[j][i] = hh < n_heads && c < n ? *reinterpret_cast<const float4*>(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    float qf = a.scale;
    if (a.temp_every > 0) qf *= fmaf(a.temp_coef, logf((float)((pos + 1) / a.temp_every + 1)), 1.f);
#pragma unroll
    for (int j = 0; j < NH; ++j) {
        const int hh = hh0 + j, kind = hh < a.H ? 0 : hh < a.H + a.G ? 1 : 2, h = kind == 0 ? hh : (hh - a.H) % a.G, n = kind == 2 ? a.vdim : a.dim;
        if (hh >= n_heads) break;
        const float* gain = kind == 0 ? a.q_gain : kind == 1 ? a.k_gain : nullptr;
        float f = 1.f;
        if (kind < 2 && a.qk_norm) {
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < NV; ++i) ss += v[j][i].x * v[j][i].x + v[j][i].y * v[j][i].y + v[j][i].z * v[j][i].z + v[j][i].w * v[j][i].w;
            f = 1.f / sqrtf(warp_sum(ss) / (float)n + a.eps);
        }
        if (kind == 0) f *= qf;
        const int padded = (kind == 2 ? v_blocks : key_blocks) * 64;
        __nv_bfloat16* dst = kind == 0 ? q16 + ((size_t)t * a.H + h) * padded
                                       : cache + ((size_t)page * a.G + h) * (size_t)(key_blocks + v_blocks) * (kKvTile * 64) +
                                             (kind == 2 ? (size_t)key_blocks * (kKvTile * 64) : 0);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (i * 32 + lane) * 4;
            if (c >= padded) continue;
            float4 g = make_float4(f, f, f, f);
            if (gain && c < n) {
                const float4 w = *reinterpret_cast<const float4*>(gain + c);
                g = make_float4(w.x * f, w.y * f, w.z * f, w.w * f);
            }
            *reinterpret_cast<uint2*>(dst + (kind == 0 ? c : latent_chunk16(pos % kKvTile, c >> 3) + (c & 7))) =
                make_uint2(pack_bf16(v[j][i].x * g.x, v[j][i].y * g.y), pack_bf16(v[j][i].z * g.z, v[j][i].w * g.w));
        }
    }
}

// ------------------------------------------------------------------ single tokens
// The factor that finishes a row whose softmax maximum is m and sum l: the sink's term, the head's gate, the division.
__device__ __forceinline__ float paged16_finish(float m, float l, const Paged16Args& a, int t, int h) {
    float g = 1.f;
    if (a.sink) {
        // relative to the larger of m and the sink, so that neither exponential overflows
        const float s = a.sink[h], top = fmaxf(m, s);
        g = expf(m - top);
        l = l * g + expf(s - top);
    }
    if (a.gate && !a.gate_wide) g *= sigmoid_full(a.gate[(size_t)t * a.ldg + h]);
    return g / l;
}
__device__ __forceinline__ void paged16_put(const Paged16Args& a, int t, int h, int c, float v) {
    if (a.gate && a.gate_wide) v *= sigmoid_full(a.gate[(size_t)t * a.ldg + (size_t)h * a.vdim + c]);
    const size_t at = ((size_t)t * a.H + h) * a.vdim + c;
    if (a.out_hi) {
        const __nv_bfloat16 hi = __float2bfloat16_rn(v);
        ((__nv_bfloat16*)a.out_hi)[at] = hi;
        ((__nv_bfloat16*)a.out_lo)[at] = __float2bfloat16_rn(v - __bfloat162float(hi));
    } else {
        a.out[at] = v;
    }
}

// mma.sync m16n8k16, bf16 operands, fp32 accumulation and softmax: one CTA per (token, key share, key head with 16 of its query
// heads and, for values beyond 256 columns, group of value columns).  The query heads are the M rows of every product, so all rows
// of a tile see the same keys and one mask.  Each of the four warps takes every fourth 16-key tile of the share: the tile is copied
// into the warp's own double buffer with cp.async one tile ahead, S = Q K^T (ldmatrix fragments of Q and of the tile), online
// softmax in registers, O += P V with the value columns read through ldmatrix.trans — the key columns themselves where the two are
// one array.  The warps' (max, sum, O) are merged through shared memory.
// A tile's row in shared memory: kp 32-column pieces of keys, then (values apart) the CTA's value pieces.  vc value pieces in all; a
// CTA sums VC <= 8 of them (O is 4 * VC accumulator tiles per thread); the last may hold columns nobody reads.
__device__ __forceinline__ void cp_async16(void* dst_smem, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst_smem)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_1() { asm volatile("cp.async.wait_group 1;" ::: "memory"); }

template <int VC>
__global__ void __launch_bounds__(128) paged16_mma_kernel(Paged16Args a, int kp, int vc, int row_groups, int v_groups, int n_split) {
    const bool apart = a.v_block > 0;
    const int grp = a.H / a.G;
    const int g = blockIdx.z / (row_groups * v_groups), rest = blockIdx.z % (row_groups * v_groups);
    const int r0 = (rest % row_groups) * 16, v_first = (rest / row_groups) * VC;      // first query head of the group, first value piece
    const int nch = 4 * kp + (apart ? 4 * VC : 0);         // 16-byte pieces of a row
    const int RS = nch * 16 + 16;                          // row stride: 16 bytes of padding keep ldmatrix conflict-free
    const int TILE = 16 * RS, QS = 4 * kp * 16 + 16, QTILE = 16 * QS;
    extern __shared__ __align__(16) uint8_t mma_smem[];
    uint8_t* Qs = mma_smem;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    uint8_t* kbuf = mma_smem + QTILE + (size_t)warp * 2 * TILE;
    const int t = blockIdx.x, split = blockIdx.y;
    const int vdim = a.vdim, head0 = g * grp + r0;
    const __nv_bfloat16* cache = (const __nv_bfloat16*)a.cache + (size_t)g * a.blocks * (kKvTile * 64);
    const size_t page_elems = (size_t)a.G * a.blocks * (kKvTile * 64);
    const int v_chunk0 = a.v_block * 8 + v_first * 4, v_chunks = min(4 * VC, a.blocks * 8 - v_chunk0);      // the CTA's value pieces in the page
    for (int idx = threadIdx.x; idx < 16 * 4 * kp; idx += 128) {
        const int r = idx / (4 * kp), ch = idx % (4 * kp);
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r0 + r < grp) v = *reinterpret_cast<const uint4*>(a.q + ((size_t)t * a.H + head0 + r) * (a.key_blocks * 64) + ch * 8);
        *reinterpret_cast<uint4*>(Qs + r * QS + ch * 16) = v;
    }
    __syncthreads();
    const int n_keys = a.positions[t] + 1;
    int j_lo = 0, j_hi = n_keys;
    if (n_split > 1) {
        const int share = ((n_keys + n_split - 1) / n_split + 15) / 16 * 16;
        j_lo = min(split * share, n_keys);
        j_hi = min(j_lo + share, n_keys);
    }
    const int* pt = a.page_table + (size_t)a.seq_rows[t] * a.max_pages;
    const int n_tiles = (j_hi - j_lo + 15) / 16;
    auto stage = [&](int tile, int buf) {
        const int key0 = j_lo + tile * 16;
        uint8_t* dst = kbuf + buf * TILE;
        for (int i = lane; i < 16 * nch; i += 32) {
            const int r = i / nch, ch = i % nch;
            const int j = min(key0 + r, j_hi - 1);
            const int from = ch < 4 * kp ? ch : v_chunk0 + min(ch - 4 * kp, v_chunks - 1);      // pieces past the last repeat it, unread
            cp_async16(dst + r * RS + ch * 16, cache + (size_t)pt[j / kKvTile] * page_elems + latent_chunk16(j % kKvTile, from));
        }
        cp_async_commit();
    };
    float o[4 * VC][4];
#pragma unroll
    for (int nt = 0; nt < 4 * VC; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
    float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;      // rows gq and gq + 8
    const int gq = lane >> 2, tq = lane & 3;
    const uint32_t q_addr = smem_u32(Qs) + ((lane & 7) + ((lane >> 3) & 1) * 8) * QS + (lane >> 4) * 16;
    const int v_ch = apart ? 4 * kp : 4 * v_first;                     // where the CTA's value columns start in a row
    if (warp < n_tiles) stage(warp, 0);
    for (int tile = warp, it = 0; tile < n_tiles; tile += 4, ++it) {
        const int cur = it & 1;
        if (tile + 4 < n_tiles) { stage(tile + 4, cur ^ 1); cp_async_wait_1(); }
        else cp_async_wait_all();
        __syncwarp();
        const uint32_t kb = smem_u32(kbuf + cur * TILE);
        float sc[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll 2
        for (int kk = 0; kk < kp; ++kk) {                        // 32 columns per round
            uint32_t a0[4], a1[4];
            ldmatrix_x4(q_addr + (kk * 4) * 16, a0[0], a0[1], a0[2], a0[3]);
            ldmatrix_x4(q_addr + (kk * 4 + 2) * 16, a1[0], a1[1], a1[2], a1[3]);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4(kb + (8 * j + (lane & 7)) * RS + (kk * 4 + (lane >> 3)) * 16, b0, b1, b2, b3);
                mma_bf16_16816(sc[j], a0[0], a0[1], a0[2], a0[3], b0, b1);
                mma_bf16_16816(sc[j], a1[0], a1[1], a1[2], a1[3], b2, b3);
            }
        }
        const int key0 = j_lo + tile * 16 + 2 * tq;
        float ta = -INFINITY, tb = -INFINITY;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                if (key0 + 8 * j + e >= j_hi) sc[j][e] = sc[j][2 + e] = -INFINITY;
                ta = fmaxf(ta, sc[j][e]);
                tb = fmaxf(tb, sc[j][2 + e]);
            }
        ta = fmaxf(ta, __shfl_xor_sync(0xffffffffu, ta, 1));
        ta = fmaxf(ta, __shfl_xor_sync(0xffffffffu, ta, 2));
        tb = fmaxf(tb, __shfl_xor_sync(0xffffffffu, tb, 1));
        tb = fmaxf(tb, __shfl_xor_sync(0xffffffffu, tb, 2));
        const float na = fmaxf(m_a, ta), nb = fmaxf(m_b, tb);      // finite: the tile's first key is never masked
        const float alpha_a = expf(m_a - na), alpha_b = expf(m_b - nb);
        float sa = 0.f, sb = 0.f;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                sc[j][e] = expf(sc[j][e] - na);
                sc[j][2 + e] = expf(sc[j][2 + e] - nb);
                sa += sc[j][e];
                sb += sc[j][2 + e];
            }
        l_a = l_a * alpha_a + sa;
        l_b = l_b * alpha_b + sb;
        m_a = na;
        m_b = nb;
        const uint32_t pa0 = pack_bf16(sc[0][0], sc[0][1]), pa1 = pack_bf16(sc[0][2], sc[0][3]);
        const uint32_t pa2 = pack_bf16(sc[1][0], sc[1][1]), pa3 = pack_bf16(sc[1][2], sc[1][3]);
        const int vrow = ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
        for (int np = 0; np < 2 * VC; ++np) {                    // 16 value columns per round
            if (v_first + (np >> 1) >= vc) break;                // the last group of columns may be a partial one
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(kb + vrow * RS + (v_ch + 2 * np + (lane >> 4)) * 16, b0, b1, b2, b3);
            o[2 * np][0] *= alpha_a; o[2 * np][1] *= alpha_a; o[2 * np][2] *= alpha_b; o[2 * np][3] *= alpha_b;
            o[2 * np + 1][0] *= alpha_a; o[2 * np + 1][1] *= alpha_a; o[2 * np + 1][2] *= alpha_b; o[2 * np + 1][3] *= alpha_b;
            mma_bf16_16816(o[2 * np], pa0, pa1, pa2, pa3, b0, b1);
            mma_bf16_16816(o[2 * np + 1], pa0, pa1, pa2, pa3, b2, b3);
        }
        __syncwarp();
    }
    // the warp's record in its own (now idle) buffer: 16 rows of the CTA's columns, then max and sum
    l_a += __shfl_xor_sync(0xffffffffu, l_a, 1);
    l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
    l_b += __shfl_xor_sync(0xffffffffu, l_b, 1);
    l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
    constexpr int COLS = 32 * VC, REC = COLS + 2;
    float* rec = reinterpret_cast<float*>(kbuf);
#pragma unroll
    for (int nt = 0; nt < 4 * VC; ++nt) {
        rec[gq * REC + nt * 8 + 2 * tq] = o[nt][0];
        rec[gq * REC + nt * 8 + 2 * tq + 1] = o[nt][1];
        rec[(gq + 8) * REC + nt * 8 + 2 * tq] = o[nt][2];
        rec[(gq + 8) * REC + nt * 8 + 2 * tq + 1] = o[nt][3];
    }
    if (tq == 0) {
        rec[gq * REC + COLS] = m_a; rec[gq * REC + COLS + 1] = l_a;
        rec[(gq + 8) * REC + COLS] = m_b; rec[(gq + 8) * REC + COLS + 1] = l_b;
    }
    __syncthreads();
    const int rows = min(16, grp - r0);
    for (int idx = threadIdx.x; idx < rows * COLS; idx += 128) {
        const int r = idx / COLS, c = idx % COLS, col = 32 * v_first + c;
        if (col >= vdim) continue;
        float m = -INFINITY;
#pragma unroll
        for (int w = 0; w < 4; ++w) m = fmaxf(m, reinterpret_cast<const float*>(mma_smem + QTILE + (size_t)w * 2 * TILE)[r * REC + COLS]);
        float l = 0.f, v = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float* rw = reinterpret_cast<const float*>(mma_smem + QTILE + (size_t)w * 2 * TILE) + r * REC;
            if (rw[COLS] > -INFINITY) {
                const float f = expf(rw[COLS] - m);
                l = fmaf(rw[COLS + 1], f, l);
                v = fmaf(rw[c], f, v);
            }
        }
        if (n_split > 1) {
            float* p = a.part + (((size_t)t * a.H + head0 + r) * n_split + split) * (vdim + 2);
            p[2 + col] = v;
            if (col == 0) { p[0] = m; p[1] = l; }
        } else {
            paged16_put(a, t, head0 + r, col, v * paged16_finish(m, l, a, t, head0 + r));
        }
    }
}

// The shares of one (token, head) put together: one CTA each.
__global__ void __launch_bounds__(128) paged16_merge_kernel(Paged16Args a, int n_split) {
    __shared__ float share[kAttnMaxSplits];                // what a share's sums count in the result
    const int pair = blockIdx.x, n = a.vdim, t = pair / a.H, h = pair % a.H;
    const float* p = a.part + (size_t)pair * n_split * (n + 2);
    if (threadIdx.x < 32) {
        const int s = threadIdx.x;
        const float ms = s < n_split ? p[(size_t)s * (n + 2)] : -INFINITY;
        const float m = warp_max(ms);
        const float w = ms > -INFINITY ? expf(ms - m) : 0.f;
        const float l = warp_sum(w > 0.f ? p[(size_t)s * (n + 2) + 1] * w : 0.f);
        if (s < n_split) share[s] = w * paged16_finish(m, l, a, t, h);
    }
    __syncthreads();
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
        float v = 0.f;
#pragma unroll
        for (int s = 0; s < kAttnMaxSplits; ++s)
            if (s < n_split && share[s] > 0.f) v = fmaf(p[(size_t)s * (n + 2) + 2 + c], share[s], v);
        paged16_put(a, t, h, c, v);
    }
}

struct MmaCfg { int kp, vc, per, v_groups; size_t smem; };
MmaCfg mma_cfg(const Paged16Args& a) {
    MmaCfg c;
    c.kp = a.v_block > 0 ? (a.dim + 31) / 32 : a.key_blocks * 2;
    c.vc = (a.vdim + 31) / 32;
    c.v_groups = (c.vc + 7) / 8;
    c.per = (c.vc + c.v_groups - 1) / c.v_groups;
    // the query tile, four double-buffered key tiles
    c.smem = (size_t)16 * (4 * c.kp * 16 + 16) + (size_t)8 * 16 * ((4 * c.kp + (a.v_block > 0 ? 4 * c.per : 0)) * 16 + 16);
    return c;
}

}  // namespace

bool paged16_write_ok(const WindowArgs& a) {
    return a.window == 0 && a.softcap == 0.f && !a.rel && a.keep_first == 0 && a.qk_norm <= 1 && a.o_v >= 0 && a.v_role == 0 && a.v_in_key < 0 &&
           !a.no_kv;
}

int launch_paged16_write(const WindowArgs& a, __nv_bfloat16* q16, void* cache, int T, cudaStream_t stream) {
    FT_REQUIRE(paged16_write_ok(a) && q16 && cache && a.rot_dims <= a.dim && (a.rot_dims & 1) == 0, "paged bf16 cache: attention options it does not take");
    const int kb = (a.dim + 63) / 64, vb = (a.vdim + 63) / 64, row = std::max(kb, vb) * 64;
    auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    if (a.rot_dims == 0 && !a.q_bias && !a.k_bias && !a.v_bias && a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ldp % 4 == 0 && a.o_q % 4 == 0 &&
        a.o_k % 4 == 0 && a.o_v % 4 == 0 && al(a.proj) && al(a.q_gain) && al(a.k_gain) && row <= 512) {
        const int nh = T >= 256 ? 2 : 1;
        const dim3 grid(T, (a.H + 2 * a.G + PW_WARPS * nh - 1) / (PW_WARPS * nh));
#define FT_P16W(NV_)                                                                                                                      \
    do {                                                                                                                                  \
        if (nh == 2) paged16_write_rows_kernel<NV_, 2><<<grid, PW_WARPS * 32, 0, stream>>>(a, q16, (__nv_bfloat16*)cache, kb, vb);        \
        else paged16_write_rows_kernel<NV_, 1><<<grid, PW_WARPS * 32, 0, stream>>>(a, q16, (__nv_bfloat16*)cache, kb, vb);                \
    } while (0)
        if (row <= 128) FT_P16W(1);
        else if (row <= 256) FT_P16W(2);
        else FT_P16W(4);
#undef FT_P16W
        FT_CHECK_CUDA(cudaGetLastError());
        return 0;
    }
    const size_t smem = (size_t)PW_WARPS * row * 4;
    FT_REQUIRE(smem <= 48 * 1024, "paged bf16 cache: head sizes %d / %d are too large", a.dim, a.vdim);
    const dim3 grid(T, (a.H + 2 * a.G + PW_WARPS - 1) / PW_WARPS);
    paged16_write_kernel<<<grid, PW_WARPS * 32, smem, stream>>>(a, q16, (__nv_bfloat16*)cache, kb, vb, row);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

bool paged16_mma_ok(const Paged16Args& a) {
    return a.H >= 1 && a.G >= 1 && a.H % a.G == 0 && a.dim >= 1 && a.vdim >= 1 && mma_cfg(a).smem <= 224 * 1024;
}

int launch_paged16_merge(const Paged16Args& a, int n_pairs, int n_split, cudaStream_t stream) {
    paged16_merge_kernel<<<n_pairs, 128, 0, stream>>>(a, n_split);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

int launch_paged16_mma(const Paged16Args& a, int T, cudaStream_t stream) {
    FT_REQUIRE(a.q && a.cache && paged16_mma_ok(a), "paged attention: sizes %d + %d do not fit", a.dim, a.vdim);
    const MmaCfg c = mma_cfg(a);
    const int rg = (a.H / a.G + 15) / 16;
    int n_split = a.part ? attn_splits(T, a.H) : 1;
    if (a.G > 1) {                       // several key heads: shares for about one wave of CTAs
        const long long wave = 148LL * std::max<size_t>(1, std::min<size_t>(8, (227 * 1024) / (c.smem + 1024)));
        n_split = (int)std::max<long long>(1, std::min<long long>(n_split, wave / std::max<long long>(1, (long long)T * a.G * rg * c.v_groups)));
    }
    const dim3 grid(T, n_split, a.G * rg * c.v_groups);
    FT_REQUIRE(grid.z <= 65535, "paged attention: %d heads are too many", a.H);
#define FT_P16M(VC_)                                                                                                        \
    case VC_: {                                                                                                             \
        static PerDeviceFlag attr;                                                                                          \
        if (!attr.done()) {                                                                                                 \
            FT_CHECK_CUDA(cudaFuncSetAttribute(paged16_mma_kernel<VC_>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024)); \
            attr.mark();                                                                                                    \
        }                                                                                                                   \
        paged16_mma_kernel<VC_><<<grid, 128, c.smem, stream>>>(a, c.kp, c.vc, rg, c.v_groups, n_split);                     \
        break;                                                                                                              \
    }
    switch (c.per) {
        FT_P16M(1) FT_P16M(2) FT_P16M(3) FT_P16M(4) FT_P16M(5) FT_P16M(6) FT_P16M(7) FT_P16M(8)
        default: break;
    }
#undef FT_P16M
    FT_CHECK_CUDA(cudaGetLastError());
    return n_split > 1 ? launch_paged16_merge(a, T * a.H, n_split, stream) : 0;
}

}  // namespace ft
