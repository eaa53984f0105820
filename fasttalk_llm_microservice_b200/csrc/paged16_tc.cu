// Softmax attention of prompt portions over the paged bf16 cache (Paged16Args) on tcgen05 / TMEM.
//
// The query rows of a portion that read one key head are its (token, head of the group) pairs, token-major: they all read the same
// keys, so 128 consecutive pairs are the M rows of one tile whatever the number of heads.  One CTA = one such tile of a run of 64
// tokens of a request (128 tokens where 64 would leave a tile half empty) and one key head (and, for values beyond 256 columns, one
// group of value columns).  Keys come page by page: a (page, key head) of the cache is [64-column block][64 tokens][64 columns]
// with the 16-byte chunks of a row XOR-swizzled by the token, which as it lies is the K-major 128-byte-swizzled operand of the
// scores and, block by block, the MN-major one of the values — bulk copies, no rearrangement; where the values are columns of the
// keys (latent attention) ONE array in shared memory serves both products.
//
//   S  = Q K^T   tcgen05.mma  M128 N64, over all key columns.  Q sits in TENSOR MEMORY as far as there is room (4 or
//                8 blocks of 64 columns): with both operands in shared memory an M128 N64 product asks for more than the port's
//                128 B/clk.  Further blocks lie in shared memory.
//   softmax      4 warps, one thread per row, running maximum and sum in fp32, exp2; the rescale of O is lazy (the reference
//                maximum moves only when it is exceeded by more than 2^8), P -> bf16 -> TMEM over the scores it came from
//   O += P V     tcgen05.mma  M128 N64..256, the value blocks of the same page
//
// Scores have two buffers: the product of tile j + 2 is queued right behind P V of tile j and runs while tile j + 1 is in the
// softmax.  TMEM: O 256 columns, S 2 x 64, Q 128 (+ 128 of O's when a value has at most 128 columns).
// Heads of at most 128 columns leave room for TWO CTAs per SM, which hide each other's waits better than a second buffer does:
// TMEM O 128, S 64, Q 64 each.
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
constexpr int LT_COL_O = 0;
// TMEM columns and score buffers of the two forms: one CTA per SM (512 columns), two (256 columns)
template <int PER_SM> struct LtTmem { static constexpr int COLS = 512, S = 256, Q = 384, Q2 = 128, NBUF = 2, QB = 5; };
template <> struct LtTmem<2> { static constexpr int COLS = 256, S = 128, Q = 192, Q2 = 0, NBUF = 1, QB = 2; };
constexpr float LT_RESCALE = 8.f;                      // log2 units
constexpr float LOG2E = 1.4426950408889634f;
constexpr int LT_OUT_LD = 36;                          // floats per row of a warp's output staging (32 columns)
constexpr size_t LT_SMEM_MAX = 227 * 1024;

struct PagedTcCfg {
    int nblk, tq, stages, nv, groups;                  // key blocks, blocks of Q in TMEM, ring, value columns per CTA, groups of them
    int sblk;                                          // blocks of one stage: the keys and, where they are apart, the CTA's values
    int span, grp;                                     // tokens per run, query heads per key head
    int per_sm;                                        // CTAs per SM
    size_t smem;
};

bool paged_tc_cfg(const Paged16Args& a, PagedTcCfg& c) {
    const int vblk = (a.vdim + 63) / 64;
    c.nblk = a.key_blocks;
    c.groups = (vblk + 3) / 4;
    c.nv = (vblk + c.groups - 1) / c.groups * 64;
    c.tq = std::min(c.nblk, c.nv <= 128 ? 8 : 4);
    c.sblk = c.nblk + (a.v_block > 0 ? c.nv / 64 : 0);
    c.grp = a.G > 0 ? std::max(a.H / a.G, 1) : 1;
    c.span = c.grp % 2 == 0 ? kKvTile : 2 * kKvTile;
    c.per_sm = c.nblk <= 2 && c.groups == 1 && c.nv <= 128 ? 2 : 1;
    const size_t fixed = 1024 + (size_t)(c.nblk - c.tq) * LT_QBLK + 256, room = c.per_sm == 2 ? 112 * 1024 : LT_SMEM_MAX;
    if (fixed >= room) return false;
    c.stages = (int)std::min<size_t>(LT_MAX_STAGES, (room - fixed) / ((size_t)c.sblk * LT_SLAB));
    c.smem = fixed + (size_t)std::max(c.stages, 0) * c.sblk * LT_SLAB;
    return c.stages >= 2;
}

template <int PER_SM>
__global__ void __launch_bounds__(LT_THREADS, PER_SM)
paged16_tc_kernel(Paged16Args a, WindowTiles tm, PagedTcCfg cfg, int subs, int* err) {
    using TM = LtTmem<PER_SM>;
    constexpr int NBUF = TM::NBUF;                                     // score buffers
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int stage_bytes = cfg.sblk * LT_SLAB;
    uint8_t* kv_s = smem;                                              // [stages][sblk] slabs
    uint8_t* q_s = kv_s + (size_t)cfg.stages * stage_bytes;             // blocks of Q that TMEM has no room for
    uint64_t* kv_full = reinterpret_cast<uint64_t*>(q_s + (size_t)(cfg.nblk - cfg.tq) * LT_QBLK);      // [6]
    uint64_t* kv_empty = kv_full + LT_MAX_STAGES;                      // [6] the products of the page have retired: O holds its share
    uint64_t* q_full = kv_empty + LT_MAX_STAGES;
    uint64_t* s_full = q_full + 1;                                     // [2]
    uint64_t* p_full = s_full + 2;                                     // [2]
    uint64_t* drain = p_full + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(drain + 1);
    volatile int* dead = reinterpret_cast<volatile int*>(tmem_slot + 1);

    // the last tiles of a request see the most keys: they go first
    const int lin = ((int)gridDim.x - 1 - (int)blockIdx.x) / a.G, tile = lin / subs, sub = lin % subs, kv_head = blockIdx.x % a.G;
    const int req = tm.tile_req[tile], q0 = tm.tile_q0[tile];
    if (q0 % cfg.span != 0) return;                                    // a run of two query tiles belongs to the first of them
    const int row0 = tm.req_q_start[req] + q0, p0 = tm.req_pos0[req] + q0;
    const int grp = cfg.grp, head0 = kv_head * grp;
    const int ntok = min(cfg.span, tm.req_q_start[req + 1] - row0);
    const int first = sub * LT_ROWS;                                   // first (token, head) pair of this tile
    if (first >= ntok * grp) return;
    const int last_tok = min((first + LT_ROWS - 1) / grp, ntok - 1);
    const int n_tiles = (p0 + last_tok) / kKvTile + 1;
    const int v0 = blockIdx.y * cfg.nv;                                // first value column
    const bool apart = a.v_block > 0;                                  // values in blocks of their own
    const int nv = min(cfg.nv, (a.vdim + 63) / 64 * 64 - v0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        for (int s = 0; s < cfg.stages; ++s) { mbar_init(&kv_full[s], 1); mbar_init(&kv_empty[s], 1); }
        mbar_init(q_full, LT_ROWS / 32);
        for (int b = 0; b < 2; ++b) {
            mbar_init(&s_full[b], 1);
            mbar_init(&p_full[b], LT_ROWS / 32);
        }
        mbar_init(drain, 1);
        *dead = 0;
        fence_mbar_init();
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, TM::COLS);
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
                    ok = mbar_wait_limited(&kv_empty[s], (round & 1) ^ 1, dead);
                    if (ok) {
                        const uint8_t* src = (const uint8_t*)a.cache + ((size_t)page * a.G + kv_head) * a.blocks * LT_SLAB;
                        uint8_t* dst = kv_s + (size_t)s * stage_bytes;
                        const int kb = cfg.nblk * LT_SLAB, vb = apart ? nv * (LT_SLAB / 64) : 0;
                        mbar_expect_tx(&kv_full[s], kb + vb);
                        tma_bulk_g2s(dst, src, kb, &kv_full[s], pol);
                        if (apart) tma_bulk_g2s(dst + kb, src + (size_t)(a.v_block + (v0 >> 6)) * LT_SLAB, vb, &kv_full[s], pol);
                        ++issued;
                    }
                }
                ok = __shfl_sync(0xffffffffu, (int)ok, 0) != 0;
            }
        }
        if (!ok && lane == 0)                                          // copies in flight land before the CTA's memory goes away
            for (int k = max(0, issued - cfg.stages); k < issued; ++k)
                for (int i = 0; i < kWaitLimit && !mbar_try_wait(&kv_full[k % cfg.stages], (k / cfg.stages) & 1); ++i) {}
    } else if (warp == 1) {
        // ---------------------------------------------------------------- products
        if (elect_one()) {
            const uint32_t idesc_qk = umma_idesc_bf16(LT_ROWS, kKvTile);
            const uint32_t idesc_pv = umma_idesc_bf16(LT_ROWS, nv) | (1u << 16);      // B is MN-major
            const uint32_t kv_addr = smem_u32(kv_s), q_addr = smem_u32(q_s);
            auto stage_at = [&](int j) { return kv_addr + (uint32_t)(j % cfg.stages) * stage_bytes; };
            auto issue_qk = [&](int j) {
                const uint32_t k_addr = stage_at(j), d = tmem + TM::S + (j % NBUF) * 64;
                uint64_t b = umma_desc_k128(k_addr);
                uint32_t acc = 0;
                // whole blocks: columns beyond the row's end are zeros on both sides.  Little besides the products in here: one
                // thread issues them all
                for (int blk = 0; blk < cfg.tq; ++blk, b += LT_SLAB >> 4) {
                    const uint32_t qa = tmem + (blk < 4 ? TM::Q : TM::Q2 - 128) + 32 * blk;
#pragma unroll
                    for (int k = 0; k < 4; ++k) { umma_f16_ts(d, qa + 8 * k, b + 2 * k, idesc_qk, acc); acc = 1; }
                }
                uint64_t qd = umma_desc_k128(q_addr);
                for (int blk = cfg.tq; blk < cfg.nblk; ++blk, b += LT_SLAB >> 4, qd += LT_QBLK >> 4) {
#pragma unroll
                    for (int k = 0; k < 4; ++k) umma_bf16(d, qd + 2 * k, b + 2 * k, idesc_qk, 1);
                }
                umma_commit(&s_full[j % NBUF]);
            };
            bool ok = mbar_wait_limited(q_full, 0, dead);
            tc_fence_after();
            for (int j = 0; j < NBUF && j < n_tiles && ok; ++j) {
                ok = mbar_wait_limited(&kv_full[j % cfg.stages], (j / cfg.stages) & 1, dead);
                tc_fence_after();
                if (ok) issue_qk(j);
            }
            const bool ahead = cfg.stages > NBUF;                      // page j + NBUF does not wait for the products of page j
            for (int j = 0; j < n_tiles && ok; ++j) {
                if (ahead && j + NBUF < n_tiles) ok = mbar_wait_limited(&kv_full[(j + NBUF) % cfg.stages], ((j + NBUF) / cfg.stages) & 1, dead);
                ok = ok && mbar_wait_limited(&p_full[j % NBUF], (j / NBUF) & 1, dead);      // P(j) written, S(j) consumed, O rescaled if needed
                if (!ok) break;
                tc_fence_after();
                const uint32_t p = tmem + TM::S + (j % NBUF) * 64, v_addr = stage_at(j) + (apart ? cfg.nblk : v0 >> 6) * LT_SLAB;
                const uint64_t vd = umma_desc_mn128(v_addr);
#pragma unroll
                for (int k = 0; k < kKvTile / 16; ++k)
                    umma_f16_ts(tmem + LT_COL_O, p + 8 * k, vd + k * (2048 >> 4), idesc_pv, (j | k) != 0);
                umma_commit(&kv_empty[j % cfg.stages]);
                if (j + NBUF < n_tiles) {
                    if (!ahead) ok = mbar_wait_limited(&kv_full[(j + NBUF) % cfg.stages], ((j + NBUF) / cfg.stages) & 1, dead);
                    tc_fence_after();
                    if (ok) issue_qk(j + NBUF);                           // behind the product that reads P out of this buffer
                }
            }
            if (!ok) {
                umma_commit(drain);
                for (int i = 0; i < kWaitLimit && !mbar_try_wait(drain, 0); ++i) {}
            }
        }
    } else {
        // ---------------------------------------------------------------- queries in, softmax, results out (one thread per row)
        const int quarter = warp & 3, row = quarter * 32 + lane;       // TMEM lane == row
        const int pair = first + row, tok = pair / grp, head = head0 + pair % grp;
        const bool valid = tok < ntok;
        const int pos = valid ? p0 + tok : p0 + last_tok;
        const uint32_t lanes = tmem + ((uint32_t)(quarter * 32) << 16);
        const uint4* q = reinterpret_cast<const uint4*>(a.q + ((size_t)(row0 + (valid ? tok : 0)) * a.H + head) * (cfg.nblk * 64));
        constexpr int QB = TM::QB;                                        // blocks of a row on their way at a time
        for (int b0 = 0; b0 < cfg.nblk; b0 += QB) {
            uint4 v[QB][8];
#pragma unroll
            for (int i = 0; i < QB; ++i)
#pragma unroll
                for (int ch = 0; ch < 8; ++ch) v[i][ch] = valid && b0 + i < cfg.nblk ? q[(b0 + i) * 8 + ch] : make_uint4(0u, 0u, 0u, 0u);
            __syncwarp();
#pragma unroll
            for (int i = 0; i < QB; ++i) {
                const int blk = b0 + i;
                if (blk < cfg.tq) {
                    const uint32_t dst = lanes + (blk < 4 ? TM::Q : TM::Q2 - 128) + 32 * blk;
                    tmem_st16(dst, &v[i][0].x);
                    tmem_st16(dst + 16, &v[i][4].x);
                } else if (blk < cfg.nblk) {
                    uint8_t* dst = q_s + (size_t)(blk - cfg.tq) * LT_QBLK + row * 128;
#pragma unroll
                    for (int ch = 0; ch < 8; ++ch) *reinterpret_cast<uint4*>(dst + ((ch ^ (row & 7)) << 4)) = v[i][ch];
                }
            }
        }
        tmem_st_wait();
        fence_proxy_async();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(q_full);
        if (a.gate && a.gate_wide && valid)                            // the row's gate values on their way to L2 meanwhile
            for (int c = 0; c < nv && v0 + c < a.vdim; c += 32)
                asm volatile("prefetch.global.L2 [%0];" ::"l"(a.gate + (size_t)(row0 + tok) * a.ldg + (size_t)head * a.vdim + v0 + c));

        float m_ref = -INFINITY, l_run = 0.f;                          // log2 units
        bool ok = true;
        for (int j = 0; j < n_tiles; ++j) {
            ok = __all_sync(0xffffffffu, mbar_wait_limited(&s_full[j % NBUF], (j / NBUF) & 1, dead));
            if (!ok) break;
            tc_fence_after();
            const uint32_t s_addr = lanes + TM::S + (j % NBUF) * 64;
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
            const float m_new = fmaxf(m_ref, fmaxf(fmaxf(t4[0], t4[1]), fmaxf(t4[2], t4[3])) * LOG2E);
            if (j == 0) {
                m_ref = m_new;                                         // finite: position 0 is visible to every row
            } else if (__any_sync(0xffffffffu, m_new > m_ref + LT_RESCALE)) {      // tcgen05.ld / st move whole warps
                ok = __all_sync(0xffffffffu, mbar_wait_limited(&kv_empty[(j - 1) % cfg.stages], ((j - 1) / cfg.stages) & 1, dead));
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
                    const float x = ex2_fast(fmaf(__uint_as_float(sr[half * 32 + 2 * e]), LOG2E, -m_ref));
                    const float y = ex2_fast(fmaf(__uint_as_float(sr[half * 32 + 2 * e + 1]), LOG2E, -m_ref));
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
            if (lane == 0) mbar_arrive(&p_full[j % NBUF]);
        }
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait_limited(&kv_empty[(n_tiles - 1) % cfg.stages], ((n_tiles - 1) / cfg.stages) & 1, dead));
        if (ok) {
            tc_fence_after();
            float f = 1.f;
            if (a.sink && valid) {                                     // relative to the larger of maximum and sink
                const float s = a.sink[head] * LOG2E, top = fmaxf(m_ref, s);
                f = exp2f(m_ref - top);
                l_run = l_run * f + exp2f(s - top);
            }
            if (a.gate && !a.gate_wide && valid) f *= 1.f / (1.f + expf(-a.gate[(size_t)(row0 + tok) * a.ldg + head]));
            f /= l_run;
            // 32 columns at a time through shared memory (the ring is idle now), so that a store covers whole 128-byte runs
            float* stage = reinterpret_cast<float*>(kv_s) + quarter * 32 * LT_OUT_LD;
            const int rows = min(32, ntok * grp - first - quarter * 32);      // valid rows of this warp (may be <= 0)
            const bool v4 = (a.vdim & 3) == 0 && (a.ldg & 3) == 0;
            __nv_bfloat16 *hi = (__nv_bfloat16*)a.out_hi, *lo = (__nv_bfloat16*)a.out_lo;
            const bool wide = a.gate && a.gate_wide;
            // where this lane's eight rows (every fourth) lie in the result and in the gate, from the run's first row
            const size_t out0 = (size_t)row0 * a.H * a.vdim, gate0 = (size_t)row0 * a.ldg;
            int at[8], gat[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int pr = first + quarter * 32 + i * 4 + (lane >> 3), t = pr / grp, h = head0 + pr - t * grp;
                at[i] = (t * a.H + h) * a.vdim;
                gat[i] = t * a.ldg + h * a.vdim;
            }
            for (int c = 0; c < nv && v0 + c < a.vdim; c += 32) {
                const int k = (lane & 7) * 4, col = v0 + c + k;               // the four columns this lane stores, of every fourth row
                float4 g[8];
                if (wide) {
#pragma unroll
                    for (int i = 0; i < 8; ++i) {                             // all gate values on the way before the first is used
                        g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                        if (i * 4 + (lane >> 3) < rows && col < a.vdim) {
                            const float* gp = a.gate + gate0 + gat[i] + col;
                            if (v4) g[i] = *reinterpret_cast<const float4*>(gp);
                            else {
                                g[i].x = gp[0];
                                if (col + 1 < a.vdim) g[i].y = gp[1];
                                if (col + 2 < a.vdim) g[i].z = gp[2];
                                if (col + 3 < a.vdim) g[i].w = gp[3];
                            }
                        }
                    }
                }
                uint32_t o[32];
                __syncwarp();
                tmem_ld16_nowait(lanes + LT_COL_O + c, o);
                tmem_ld16_nowait(lanes + LT_COL_O + c + 16, o + 16);
                tmem_ld_wait();
#pragma unroll
                for (int q4 = 0; q4 < 32; q4 += 4)
                    *reinterpret_cast<float4*>(stage + lane * LT_OUT_LD + q4) =
                        make_float4(__uint_as_float(o[q4]) * f, __uint_as_float(o[q4 + 1]) * f, __uint_as_float(o[q4 + 2]) * f, __uint_as_float(o[q4 + 3]) * f);
                __syncwarp();
                if (v4) {
                    float4 v[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) v[i] = *reinterpret_cast<const float4*>(stage + (i * 4 + (lane >> 3)) * LT_OUT_LD + k);
                    if (wide) {
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            v[i].x *= sigmoid_quick(g[i].x); v[i].y *= sigmoid_quick(g[i].y);
                            v[i].z *= sigmoid_quick(g[i].z); v[i].w *= sigmoid_quick(g[i].w);
                        }
                    }
                    if (hi) {
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            const uint32_t h0 = pack_bf16(v[i].x, v[i].y), h1 = pack_bf16(v[i].z, v[i].w);
                            const uint32_t l0 = pack_bf16(v[i].x - bf16_lo(h0), v[i].y - bf16_hi(h0)), l1 = pack_bf16(v[i].z - bf16_lo(h1), v[i].w - bf16_hi(h1));
                            if (i * 4 + (lane >> 3) < rows && col < a.vdim) {
                                *reinterpret_cast<uint2*>(hi + out0 + at[i] + col) = make_uint2(h0, h1);
                                *reinterpret_cast<uint2*>(lo + out0 + at[i] + col) = make_uint2(l0, l1);
                            }
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < 8; ++i)
                            if (i * 4 + (lane >> 3) < rows && col < a.vdim) *reinterpret_cast<float4*>(a.out + out0 + at[i] + col) = v[i];
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        const int r = i * 4 + (lane >> 3);
                        const float gv[4] = {g[i].x, g[i].y, g[i].z, g[i].w};
#pragma unroll
                        for (int q1 = 0; q1 < 4; ++q1) {
                            if (r >= rows || col + q1 >= a.vdim) continue;
                            float v = stage[r * LT_OUT_LD + k + q1];
                            if (wide) v *= sigmoid_quick(gv[q1]);
                            const size_t to = out0 + at[i] + col + q1;
                            if (hi) {
                                const __nv_bfloat16 b = __float2bfloat16_rn(v);
                                hi[to] = b;
                                lo[to] = __float2bfloat16_rn(v - __bfloat162float(b));
                            } else {
                                a.out[to] = v;
                            }
                        }
                    }
                }
                __syncwarp();
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem, TM::COLS);
    }
    if (threadIdx.x == 0 && *dead && err) *err = 1;
}

}  // namespace

bool paged16_tc_ok(const Paged16Args& a) {
    PagedTcCfg c;
    return a.H >= 1 && a.G >= 1 && a.H % a.G == 0 && a.key_blocks >= 1 && a.vdim >= 1 && paged_tc_cfg(a, c);
}

int launch_paged16_tc(const Paged16Args& a, const WindowTiles& tm, int* err, cudaStream_t stream) {
    PagedTcCfg c;
    FT_REQUIRE(a.cache && a.q && paged16_tc_ok(a) && paged_tc_cfg(a, c), "paged attention (tcgen05): sizes %d + %d do not fit", a.dim, a.vdim);
    static PerDeviceFlag attr;
    if (!attr.done()) {
        FT_CHECK_CUDA(cudaFuncSetAttribute(paged16_tc_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LT_SMEM_MAX));
        FT_CHECK_CUDA(cudaFuncSetAttribute(paged16_tc_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024));
        attr.mark();
    }
    const int subs = (c.span * c.grp + LT_ROWS - 1) / LT_ROWS;
    const dim3 grid(tm.n_tiles * subs * a.G, c.groups);
    if (c.per_sm == 2) paged16_tc_kernel<2><<<grid, LT_THREADS, c.smem, stream>>>(a, tm, c, subs, err);
    else paged16_tc_kernel<1><<<grid, LT_THREADS, c.smem, stream>>>(a, tm, c, subs, err);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace ft
