// Latent attention of prompt portions on tcgen05 / TMEM: one shared key row per token, [latent | rotated part], whose first
// columns are also its value.
//
// The query rows of a portion are its (token, head) pairs, token-major: every head reads the same keys, so 128 consecutive
// pairs are the M rows of one tile whatever the number of heads.  One CTA = one such tile of one 64-token query tile of a request
// (and, for latents beyond 256, one group of value columns).  Keys come page by page: a page of the bf16 cache is
// [64-column block][64 tokens][64 columns] with the 16-byte chunks of a row XOR-swizzled by the token, which as it lies is the
// K-major 128-byte-swizzled operand of the scores and, block by block, the MN-major one of the values — ONE bulk copy per page,
// one array in shared memory for both products.
//
//   S  = Q C^T   tcgen05.mma  M128 N64, K in steps of 16 over all columns.  Q sits in TENSOR MEMORY as far as there is room (4 or
//                8 blocks of 64 columns): with both operands in shared memory an M128 N64 product asks for more than the port's
//                128 B/clk.  Further blocks lie in shared memory.
//   softmax      4 warps, one thread per row, running maximum and sum in fp32, exp2; the rescale of O is lazy (the reference
//                maximum moves only when it is exceeded by more than 2^8), P -> bf16 -> TMEM over the scores it came from
//   O += P C     tcgen05.mma  M128 N64..256, the value columns of the same page
//
// Scores have two buffers: the product of tile j + 2 is queued right behind P V of tile j and runs while tile j + 1 is in the
// softmax.  TMEM: O 256 columns, S 2 x 64, Q 128 (+ 128 of O's when the latent has at most 128 columns).
//
// Warp roles (192 threads): 0 = page producer, 1 = TMEM owner and MMA issuer (one thread), 2..5 = query staging, softmax, epilogue.
// Every wait has a limit; a CTA whose wait runs out marks `err`, lets its copies and products finish and returns.
#include "common.cuh"
#include "ft_internal.h"

#include <algorithm>

namespace ft {
namespace {

constexpr int LT_THREADS = 192, LT_ROWS = 128;
constexpr int LT_SLAB = kKvTile * 128;                 // bytes of one [64 tokens][64 columns] block of a page
constexpr int LT_QBLK = LT_ROWS * 128;                 // bytes of one [128 rows][64 columns] block of Q in shared memory
constexpr int LT_MAX_STAGES = 6;
constexpr int LT_COL_O = 0, LT_COL_S = 256, LT_COL_Q = 384, LT_COL_Q2 = 128;
constexpr float LT_RESCALE = 8.f;                      // log2 units
constexpr int LT_SPIN = 1 << 20;
constexpr size_t LT_SMEM_MAX = 227 * 1024;

struct LatentTcCfg {
    int nblk, ksteps, tq, stages, nv, groups;          // 64-column blocks, K steps, blocks of Q in TMEM, ring, value columns per CTA
    size_t smem;
};

bool latent_tc_cfg(int rank, int rot, LatentTcCfg& c) {
    const int vblk = (rank + 63) / 64;
    c.nblk = latent_row16(rank, rot) / 64;
    c.ksteps = (rank + rot + 15) / 16;
    c.groups = (vblk + 3) / 4;
    c.nv = (vblk + c.groups - 1) / c.groups * 64;
    c.tq = std::min(c.nblk, c.nv <= 128 ? 8 : 4);
    const size_t fixed = 1024 + (size_t)(c.nblk - c.tq) * LT_QBLK + 256;
    if (fixed >= LT_SMEM_MAX) return false;
    c.stages = (int)std::min<size_t>(LT_MAX_STAGES, (LT_SMEM_MAX - fixed) / ((size_t)c.nblk * LT_SLAB));
    c.smem = fixed + (size_t)std::max(c.stages, 0) * c.nblk * LT_SLAB;
    return c.stages >= 2;
}

// false: the limit ran out here or another warp of the CTA has given up
__device__ __forceinline__ bool wait_limited(uint64_t* bar, uint32_t parity, volatile int* dead) {
    for (int i = 0; i < LT_SPIN; ++i) {
        if (mbar_try_wait(bar, parity)) return true;
        if ((i & 31) == 31 && *dead) return false;
    }
    *dead = 1;
    return false;
}

__global__ void __launch_bounds__(LT_THREADS, 1)
latent_prefill_tc_kernel(LatentArgs a, WindowTiles tm, LatentTcCfg cfg, int subs, int* err) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int page_bytes = cfg.nblk * LT_SLAB;
    uint8_t* kv_s = smem;                                              // [stages][nblk] slabs
    uint8_t* q_s = kv_s + (size_t)cfg.stages * page_bytes;             // blocks of Q that TMEM has no room for
    uint64_t* kv_full = reinterpret_cast<uint64_t*>(q_s + (size_t)(cfg.nblk - cfg.tq) * LT_QBLK);      // [6]
    uint64_t* kv_empty = kv_full + LT_MAX_STAGES;                      // [6]
    uint64_t* q_full = kv_empty + LT_MAX_STAGES;
    uint64_t* s_full = q_full + 1;                                     // [2]
    uint64_t* p_full = s_full + 2;                                     // [2]
    uint64_t* pv_done = p_full + 2;                                    // [2]
    uint64_t* drain = pv_done + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(drain + 1);
    volatile int* dead = reinterpret_cast<volatile int*>(tmem_slot + 1);

    // the last tiles of a request see the most keys: they go first
    const int lin = (int)gridDim.x - 1 - (int)blockIdx.x, tile = lin / subs, sub = lin % subs;
    const int req = tm.tile_req[tile], q0 = tm.tile_q0[tile];
    const int row0 = tm.req_q_start[req] + q0, p0 = tm.req_pos0[req] + q0;
    const int ntok = min(kKvTile, tm.req_q_start[req + 1] - row0);
    const int first = sub * LT_ROWS;                                   // first (token, head) pair of this tile
    if (first >= ntok * a.H) return;
    const int last_tok = min((first + LT_ROWS - 1) / a.H, ntok - 1);
    const int n_tiles = (p0 + last_tok) / kKvTile + 1;
    const int v0 = blockIdx.y * cfg.nv;                                // first value column
    const int nv = min(cfg.nv, cfg.nblk * 64 - v0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        for (int s = 0; s < cfg.stages; ++s) { mbar_init(&kv_full[s], 1); mbar_init(&kv_empty[s], 1); }
        mbar_init(q_full, LT_ROWS / 32);
        for (int b = 0; b < 2; ++b) {
            mbar_init(&s_full[b], 1);
            mbar_init(&p_full[b], LT_ROWS / 32);
            mbar_init(&pv_done[b], 1);
        }
        mbar_init(drain, 1);
        *dead = 0;
        fence_mbar_init();
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, 512);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;

    if (warp == 0) {
        // ---------------------------------------------------------------- pages into the ring
        const int* pt = a.page_table + (size_t)tm.req_slot[req] * a.max_pages;
        const uint64_t pol = policy_evict_last();                      // every tile of the request reads the same pages
        int issued = 0;
        bool ok = true;
        for (int t0 = 0; t0 < n_tiles && ok; t0 += 32) {
            const int my_page = t0 + lane < n_tiles ? pt[t0 + lane] : 0;
            const int n = min(32, n_tiles - t0);
            for (int i = 0; i < n && ok; ++i) {
                const int page = __shfl_sync(0xffffffffu, my_page, i);
                if (lane == 0) {
                    const int s = issued % cfg.stages, round = issued / cfg.stages;
                    ok = wait_limited(&kv_empty[s], (round & 1) ^ 1, dead);
                    if (ok) {
                        mbar_expect_tx(&kv_full[s], page_bytes);
                        tma_bulk_g2s(kv_s + (size_t)s * page_bytes, (const uint8_t*)a.cache16 + (size_t)page * page_bytes, page_bytes,
                                     &kv_full[s], pol);
                        ++issued;
                    }
                }
                ok = __shfl_sync(0xffffffffu, (int)ok, 0) != 0;
            }
        }
        if (!ok && lane == 0)                                          // copies in flight land before the CTA's memory goes away
            for (int k = max(0, issued - cfg.stages); k < issued; ++k)
                for (int i = 0; i < LT_SPIN && !mbar_try_wait(&kv_full[k % cfg.stages], (k / cfg.stages) & 1); ++i) {}
    } else if (warp == 1) {
        // ---------------------------------------------------------------- products
        if (elect_one()) {
            const uint32_t idesc_qk = umma_idesc_bf16(LT_ROWS, kKvTile);
            const uint32_t idesc_pv = umma_idesc_bf16(LT_ROWS, nv) | (1u << 16);      // B is MN-major
            const uint32_t kv_addr = smem_u32(kv_s), q_addr = smem_u32(q_s);
            auto stage_at = [&](int j) { return kv_addr + (uint32_t)(j % cfg.stages) * page_bytes; };
            auto issue_qk = [&](int j) {
                const uint32_t k_addr = stage_at(j), d = tmem + LT_COL_S + (j & 1) * 64;
                for (int s = 0; s < cfg.ksteps; ++s) {
                    const int blk = s >> 2, k = s & 3;
                    const uint64_t b = umma_desc_k128(k_addr + blk * LT_SLAB) + 2 * k;
                    if (blk < cfg.tq) {
                        const uint32_t qa = tmem + (blk < 4 ? LT_COL_Q + 32 * blk : LT_COL_Q2 + 32 * (blk - 4)) + 8 * k;
                        umma_f16_ts(d, qa, b, idesc_qk, s != 0);
                    } else {
                        umma_bf16(d, umma_desc_k128(q_addr + (blk - cfg.tq) * LT_QBLK) + 2 * k, b, idesc_qk, s != 0);
                    }
                }
                umma_commit(&s_full[j & 1]);
            };
            bool ok = wait_limited(q_full, 0, dead);
            tc_fence_after();
            for (int j = 0; j < 2 && j < n_tiles && ok; ++j) {
                ok = wait_limited(&kv_full[j % cfg.stages], (j / cfg.stages) & 1, dead);
                tc_fence_after();
                if (ok) issue_qk(j);
            }
            for (int j = 0; j < n_tiles && ok; ++j) {
                ok = wait_limited(&p_full[j & 1], (j >> 1) & 1, dead);      // P(j) written, S(j) consumed, O rescaled if needed
                if (!ok) break;
                tc_fence_after();
                const uint32_t p = tmem + LT_COL_S + (j & 1) * 64, v_addr = stage_at(j) + (v0 >> 6) * LT_SLAB;
#pragma unroll
                for (int k = 0; k < kKvTile / 16; ++k)
                    umma_f16_ts(tmem + LT_COL_O, p + 8 * k, umma_desc_mn128(v_addr + k * 2048), idesc_pv, (j | k) != 0);
                umma_commit(&pv_done[j & 1]);
                umma_commit(&kv_empty[j % cfg.stages]);
                if (j + 2 < n_tiles) {
                    ok = wait_limited(&kv_full[(j + 2) % cfg.stages], ((j + 2) / cfg.stages) & 1, dead);
                    tc_fence_after();
                    if (ok) issue_qk(j + 2);                           // behind the product that reads P out of this buffer
                }
            }
            if (!ok) {
                umma_commit(drain);
                for (int i = 0; i < LT_SPIN && !mbar_try_wait(drain, 0); ++i) {}
            }
        }
    } else {
        // ---------------------------------------------------------------- queries in, softmax, results out (one thread per row)
        const int quarter = warp & 3, row = quarter * 32 + lane;       // TMEM lane == row
        const int pair = first + row, tok = pair / a.H, head = pair % a.H;
        const bool valid = tok < ntok;
        const int pos = valid ? p0 + tok : p0 + last_tok;
        const int kd = a.rank + a.rot;
        const uint32_t lanes = tmem + ((uint32_t)(quarter * 32) << 16);
        const float to_log2 = a.scale * 1.4426950408889634f;
        const float* q = a.qlat + ((size_t)row0 * a.H + first + row) * kd;
        const bool vec = (kd & 3) == 0;
        for (int blk = 0; blk < cfg.nblk; ++blk) {
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                uint32_t pk[16];
#pragma unroll
                for (int e4 = 0; e4 < 8; ++e4) {
                    const int c = blk * 64 + half * 32 + 4 * e4;
                    float v[4] = {0.f, 0.f, 0.f, 0.f};
                    if (valid) {
                        if (vec) {
                            if (c < kd) {
                                const float4 t = *reinterpret_cast<const float4*>(q + c);
                                v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
                            }
                        } else {
#pragma unroll
                            for (int i = 0; i < 4; ++i) if (c + i < kd) v[i] = q[c + i];
                        }
                    }
                    pk[2 * e4] = pack_bf16(v[0] * to_log2, v[1] * to_log2);
                    pk[2 * e4 + 1] = pack_bf16(v[2] * to_log2, v[3] * to_log2);
                }
                __syncwarp();
                if (blk < cfg.tq) {
                    tmem_st16(lanes + (blk < 4 ? LT_COL_Q + 32 * blk : LT_COL_Q2 + 32 * (blk - 4)) + 16 * half, pk);
                } else {
                    uint8_t* dst = q_s + (size_t)(blk - cfg.tq) * LT_QBLK + row * 128;
#pragma unroll
                    for (int ch = 0; ch < 4; ++ch)
                        *reinterpret_cast<uint4*>(dst + (((half * 4 + ch) ^ (row & 7)) << 4)) =
                            make_uint4(pk[4 * ch], pk[4 * ch + 1], pk[4 * ch + 2], pk[4 * ch + 3]);
                }
            }
        }
        tmem_st_wait();
        fence_proxy_async();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(q_full);

        float m_ref = -INFINITY, l_run = 0.f;                          // log2 units
        bool ok = true;
        for (int j = 0; j < n_tiles; ++j) {
            ok = __all_sync(0xffffffffu, wait_limited(&s_full[j & 1], (j >> 1) & 1, dead));
            if (!ok) break;
            tc_fence_after();
            const uint32_t s_addr = lanes + LT_COL_S + (j & 1) * 64;
            uint32_t sr[64];
#pragma unroll
            for (int c = 0; c < 4; ++c) tmem_ld16_nowait(s_addr + 16 * c, sr + 16 * c);
            tmem_ld_wait();
            float t4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            if (j * kKvTile + kKvTile - 1 > pos) {                     // later keys of this page are hidden from this row
#pragma unroll
                for (int c = 0; c < 64; ++c) {
                    const float v = j * kKvTile + c <= pos ? __uint_as_float(sr[c]) : -INFINITY;
                    sr[c] = __float_as_uint(v);
                    t4[c & 3] = fmaxf(t4[c & 3], v);
                }
            } else {
#pragma unroll
                for (int c = 0; c < 64; ++c) t4[c & 3] = fmaxf(t4[c & 3], __uint_as_float(sr[c]));
            }
            const float m_new = fmaxf(m_ref, fmaxf(fmaxf(t4[0], t4[1]), fmaxf(t4[2], t4[3])));
            if (j == 0) {
                m_ref = m_new;                                         // finite: position 0 is visible to every row
            } else if (__any_sync(0xffffffffu, m_new > m_ref + LT_RESCALE)) {      // tcgen05.ld / st move whole warps
                ok = __all_sync(0xffffffffu, wait_limited(&pv_done[(j - 1) & 1], ((j - 1) >> 1) & 1, dead));
                if (!ok) break;
                tc_fence_after();
                const float alpha = exp2f(m_ref - m_new);
                l_run *= alpha;
                m_ref = m_new;
                for (int c = 0; c < nv; c += 16) {
                    uint32_t o[16];
                    tmem_ld16_nowait(lanes + LT_COL_O + c, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int k = 0; k < 16; ++k) o[k] = __float_as_uint(__uint_as_float(o[k]) * alpha);
                    tmem_st16(lanes + LT_COL_O + c, o);
                }
                tmem_st_wait();
            }
            float ps[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                uint32_t pk[16];
#pragma unroll
                for (int e = 0; e < 16; ++e) {
                    const float x = ex2_fast(__uint_as_float(sr[half * 32 + 2 * e]) - m_ref);
                    const float y = ex2_fast(__uint_as_float(sr[half * 32 + 2 * e + 1]) - m_ref);
                    ps[(2 * e) & 3] += x;
                    ps[(2 * e + 1) & 3] += y;
                    pk[e] = pack_bf16(x, y);
                }
                tmem_st16(s_addr + 16 * half, pk);                     // over the scores it came from (this row has read them)
            }
            tmem_st_wait();
            l_run += (ps[0] + ps[1]) + (ps[2] + ps[3]);
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[j & 1]);
        }
        if (ok) ok = __all_sync(0xffffffffu, wait_limited(&pv_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1, dead));
        if (ok) {
            tc_fence_after();
            float f = 1.f;
            if (a.sink && valid) {                                     // relative to the larger of maximum and sink
                const float s = a.sink[head] * 1.4426950408889634f, top = fmaxf(m_ref, s);
                f = exp2f(m_ref - top);
                l_run = l_run * f + exp2f(s - top);
            }
            if (a.o_gate >= 0 && valid) f *= 1.f / (1.f + expf(-a.proj[(size_t)(row0 + tok) * a.ldp + a.o_gate + head]));
            f /= l_run;
            float* out = a.out + ((size_t)row0 * a.H + first + row) * a.rank;
            const bool vec_o = (a.rank & 3) == 0;
            for (int c = 0; c < nv && v0 + c < a.rank; c += 16) {
                uint32_t o[16];
                __syncwarp();
                tmem_ld16_nowait(lanes + LT_COL_O + c, o);
                tmem_ld_wait();
                if (valid) {
#pragma unroll
                    for (int k = 0; k < 16; k += 4) {
                        const int col = v0 + c + k;
                        float v[4];
#pragma unroll
                        for (int i = 0; i < 4; ++i) v[i] = __uint_as_float(o[k + i]) * f;
                        if (vec_o) {
                            if (col < a.rank) *reinterpret_cast<float4*>(out + col) = make_float4(v[0], v[1], v[2], v[3]);
                        } else {
#pragma unroll
                            for (int i = 0; i < 4; ++i) if (col + i < a.rank) out[col + i] = v[i];
                        }
                    }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem, 512);
    }
    if (threadIdx.x == 0 && *dead && err) *err = 1;
}

}  // namespace

bool latent_prefill_tc_ok(int rank, int rot) {
    LatentTcCfg c;
    return latent_attn_mma_ok(rank, rot) && latent_tc_cfg(rank, rot, c);
}

int launch_latent_prefill_tc(const LatentArgs& a, const WindowTiles& tm, int* err, cudaStream_t stream) {
    LatentTcCfg c;
    FT_REQUIRE(a.cache16 && latent_tc_cfg(a.rank, a.rot, c), "latent attention (tcgen05): sizes %d + %d do not fit", a.rank, a.rot);
    static PerDeviceFlag attr;
    if (!attr.done()) {
        FT_CHECK_CUDA(cudaFuncSetAttribute(latent_prefill_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LT_SMEM_MAX));
        attr.mark();
    }
    const int subs = (kKvTile * a.H + LT_ROWS - 1) / LT_ROWS;
    const dim3 grid(tm.n_tiles * subs, c.groups);
    latent_prefill_tc_kernel<<<grid, LT_THREADS, c.smem, stream>>>(a, tm, c, subs, err);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace ft
