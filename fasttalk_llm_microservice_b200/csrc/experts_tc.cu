// The matrices of a mixture of experts on tcgen05, one launch for all experts: the (token, choice) pairs lie sorted by expert
// (seg[e] .. seg[e + 1]), every CTA takes 128 rows of one expert's matrix and up to 128 of its pairs, found from seg on the device —
// the host needs no row counts and nothing waits for it.
//
//   D[128 matrix rows x 128 pairs] in TMEM = W tile (A operand, bf16) x pair tile (B operand, the fp32 activations as bf16 hi + lo
//   planes: two products into one fp32 accumulator).  A pair tile may run over into the next expert's pairs; those columns are not stored.
//
// Epilogue by kind: fp32 rows (second matrix), or the activation — (gate, up) pairs of neighbouring rows, or squared ReLU — as bf16
// planes, the second matrix's input.  192 threads: warp 0 brings the tiles in with TMA, one thread of warp 1 issues the products,
// warps 2..5 are the epilogue.  Two stages per CTA and two CTAs per SM: one CTA's epilogue runs under the other's products.
// Every wait has a limit; a CTA whose wait runs out marks `err`, lets its copies and products finish and returns.
#include "common.cuh"
#include "ft_internal.h"

namespace ft {
namespace {

constexpr int XT_THREADS = 192, XT_M = 128, XT_N = 128, XT_K = 64, XT_STAGES = 2;
constexpr int XT_TILE = XT_M * XT_K * 2;                // bytes of one operand tile (W, hi or lo)
constexpr int XT_STAGE = 3 * XT_TILE, XT_SMEM = 1024 + XT_STAGES * XT_STAGE;
enum { XT_ROWS = 0, XT_GLU = 1, XT_RELU2 = 2 };

struct ExpertsKernelArgs {
    const int* seg;
    int E, n_rows, kb;                                  // rows of one expert's matrix, 64-column blocks of K
    GluSpec glu;
    float* out;                                         // XT_ROWS: [pair][n_rows]
    __nv_bfloat16 *hi, *lo;                             // planes [pair][n_rows / 2] (XT_GLU) or [pair][n_rows]
    int* err;
};

template <int KIND>
__global__ void __launch_bounds__(XT_THREADS, 2)
experts_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_hi, const __grid_constant__ CUtensorMap map_lo,
                  ExpertsKernelArgs a) {
    extern __shared__ uint8_t xt_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(xt_raw) + 1023) & ~uintptr_t(1023));
    __shared__ uint64_t full[XT_STAGES], empty[XT_STAGES], acc_full, drain;
    __shared__ uint32_t tmem_slot;
    __shared__ int s_tile[3];                           // expert, first pair, pairs of this tile
    __shared__ int s_dead;
    volatile int* dead = &s_dead;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (warp == 0) {
        // tile blockIdx.y of all experts' pair tiles, in order
        int before = 0, found = -1, first = 0, n = 0;
        for (int e0 = 0; e0 < a.E && found < 0; e0 += 32) {
            const int e = e0 + lane;
            const int s0 = e < a.E ? a.seg[e] : 0, s1 = e < a.E ? a.seg[e + 1] : 0, mine = (s1 - s0 + XT_N - 1) / XT_N;
            int upto = mine;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, upto, o);
                if (lane >= o) upto += v;
            }
            const unsigned hit = __ballot_sync(0xffffffffu, before + upto > (int)blockIdx.y);
            if (hit) {
                const int l = __ffs(hit) - 1;
                const int t = (int)blockIdx.y - before - __shfl_sync(0xffffffffu, upto - mine, l);
                const int b0 = __shfl_sync(0xffffffffu, s0, l), b1 = __shfl_sync(0xffffffffu, s1, l);
                found = e0 + l;
                first = b0 + t * XT_N;
                n = min(XT_N, b1 - first);
            }
            before += __shfl_sync(0xffffffffu, upto, 31);
        }
        if (lane == 0) {
            s_tile[0] = found; s_tile[1] = first; s_tile[2] = n;
            s_dead = 0;
            for (int s = 0; s < XT_STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
            mbar_init(&acc_full, 1);
            mbar_init(&drain, 1);
            fence_mbar_init();
        }
    }
    __syncthreads();
    const int expert = s_tile[0], first = s_tile[1], n = s_tile[2];
    if (expert < 0) return;                             // beyond the last tile
    if (warp == 1) {
        tmem_alloc(&tmem_slot, XT_N);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    if (warp == 0) {
        if (elect_one()) {
            tma_prefetch_desc(&map_w);
            tma_prefetch_desc(&map_hi);
            tma_prefetch_desc(&map_lo);
            const uint64_t pol_w = policy_evict_first(), pol_x = policy_evict_last();
            const int wrow = expert * a.n_rows + blockIdx.x * XT_M;
            int kb = 0;
            bool ok = true;
            for (; kb < a.kb; ++kb) {
                const int s = kb % XT_STAGES;
                ok = mbar_wait_limited(&empty[s], ((kb / XT_STAGES) & 1) ^ 1, dead);
                if (!ok) break;
                uint8_t* st = smem + (size_t)s * XT_STAGE;
                mbar_expect_tx(&full[s], XT_STAGE);
                tma_tile_2d(st, &map_w, kb * XT_K, wrow, &full[s], pol_w);
                tma_tile_2d(st + XT_TILE, &map_hi, kb * XT_K, first, &full[s], pol_x);
                tma_tile_2d(st + 2 * XT_TILE, &map_lo, kb * XT_K, first, &full[s], pol_x);
            }
            if (!ok)                                    // copies in flight land before the CTA's memory goes away
                for (int k = max(0, kb - XT_STAGES); k < kb; ++k)
                    for (int i = 0; i < kWaitLimit && !mbar_try_wait(&full[k % XT_STAGES], (k / XT_STAGES) & 1); ++i) {}
        }
    } else if (warp == 1) {
        if (elect_one()) {
            constexpr uint32_t idesc = umma_idesc_bf16(XT_M, XT_N);
            bool ok = true;
            for (int kb = 0; kb < a.kb && ok; ++kb) {
                const int s = kb % XT_STAGES;
                ok = mbar_wait_limited(&full[s], (kb / XT_STAGES) & 1, dead);
                if (!ok) break;
                tc_fence_after();
                const uint32_t base = smem_u32(smem + (size_t)s * XT_STAGE);
                const uint64_t wd = umma_desc_k128(base), hd = umma_desc_k128(base + XT_TILE), ld = umma_desc_k128(base + 2 * XT_TILE);
#pragma unroll
                for (int k = 0; k < XT_K / 16; ++k) umma_bf16(tmem, wd + 2 * k, hd + 2 * k, idesc, (kb | k) != 0);
#pragma unroll
                for (int k = 0; k < XT_K / 16; ++k) umma_bf16(tmem, wd + 2 * k, ld + 2 * k, idesc, 1u);
                umma_commit(&empty[s]);
            }
            umma_commit(ok ? &acc_full : &drain);
            if (!ok)
                for (int i = 0; i < kWaitLimit && !mbar_try_wait(&drain, 0); ++i) {}
        }
    } else {
        bool ok = __all_sync(0xffffffffu, mbar_wait_limited(&acc_full, 0, dead));
        tc_fence_after();
        const int quarter = warp & 3, et = threadIdx.x - 64;
        const uint32_t lanes = tmem + ((uint32_t)(quarter * 32) << 16);
        const int f = quarter * 32 + lane;              // row of the tile == lane of TMEM
        if (KIND == XT_ROWS) {
            if (ok) {
                float* out = a.out + (size_t)first * a.n_rows + blockIdx.x * XT_M + f;
                for (int c = 0; c < n; c += 16) {
                    float v[16];
                    __syncwarp();
                    tmem_ld16(lanes + c, v);
                    const int m = min(16, n - c);
#pragma unroll
                    for (int i = 0; i < 16; ++i)
                        if (i < m) out[(size_t)(c + i) * a.n_rows] = v[i];
                }
            }
        } else {
            // the activation's planes through shared memory (the stages are idle now): rows of pairs, then whole rows out
            constexpr int COLS = KIND == XT_GLU ? XT_M / 2 : XT_M, LD = COLS + 8;
            __nv_bfloat16 *th = reinterpret_cast<__nv_bfloat16*>(smem), *tl = th + XT_N * LD;
            auto put = [&](int pair, int col, float v) {
                const __nv_bfloat16 b = __float2bfloat16_rn(v);
                th[pair * LD + col] = b;
                tl[pair * LD + col] = __float2bfloat16_rn(v - __bfloat162float(b));
            };
            if (ok) {
                for (int c = 0; c < n; c += 16) {
                    float v[16];
                    __syncwarp();
                    tmem_ld16(lanes + c, v);
                    if (KIND == XT_GLU) {
                        // rows (2j, 2j + 1) = (gate, up) are neighbouring lanes: the even one takes eight pairs, the odd one the other eight
                        const bool odd = lane & 1;
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            const float got = __shfl_xor_sync(0xffffffffu, odd ? v[i] : v[i + 8], 1);
                            const float g = odd ? got : v[i], u = odd ? v[i + 8] : got;
                            put(c + i + (odd ? 8 : 0), f >> 1, glu_value(a.glu, g, u, blockIdx.x * (XT_M / 2) + (f >> 1)));
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i) { const float r = fmaxf(v[i], 0.f); put(c + i, f, r * r); }
                    }
                }
            }
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (ok) {
                const int ldo = KIND == XT_GLU ? a.n_rows / 2 : a.n_rows;
                for (int i = et; i < n * (COLS / 8); i += 128) {
                    const int r = i / (COLS / 8), ch = i % (COLS / 8);
                    const size_t at = (size_t)(first + r) * ldo + blockIdx.x * COLS + ch * 8;
                    *reinterpret_cast<uint4*>(a.hi + at) = *reinterpret_cast<const uint4*>(th + r * LD + ch * 8);
                    *reinterpret_cast<uint4*>(a.lo + at) = *reinterpret_cast<const uint4*>(tl + r * LD + ch * 8);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem, XT_N);
    }
    if (threadIdx.x == 0 && *dead && a.err) *a.err = 1;
}

}  // namespace

bool experts_tc_ok(int n_rows, int K) { return n_rows % XT_M == 0 && K % XT_K == 0; }

int launch_experts_tc(const ExpertsTcArgs& t, cudaStream_t stream) {
    FT_REQUIRE(t.w && t.x_hi && t.x_lo && t.seg && t.pairs >= 1 && t.E >= 1 && experts_tc_ok(t.n_rows, t.K) && (t.out || (t.out_hi && t.out_lo)),
               "experts (tcgen05): sizes or operands do not fit");
    CUtensorMap mw, mh, ml;
    if (int r = make_tmap_bf16_k64(&mw, t.w, t.E * t.n_rows, t.K, XT_M)) return r;
    if (int r = make_tmap_bf16_k64(&mh, t.x_hi, t.pairs, t.K, XT_N)) return r;
    if (int r = make_tmap_bf16_k64(&ml, t.x_lo, t.pairs, t.K, XT_N)) return r;
    static PerDeviceFlag attr;
    if (!attr.done()) {
        FT_CHECK_CUDA(cudaFuncSetAttribute(experts_tc_kernel<XT_ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, XT_SMEM));
        FT_CHECK_CUDA(cudaFuncSetAttribute(experts_tc_kernel<XT_GLU>, cudaFuncAttributeMaxDynamicSharedMemorySize, XT_SMEM));
        FT_CHECK_CUDA(cudaFuncSetAttribute(experts_tc_kernel<XT_RELU2>, cudaFuncAttributeMaxDynamicSharedMemorySize, XT_SMEM));
        attr.mark();
    }
    ExpertsKernelArgs a = {t.seg, t.E, t.n_rows, t.K / XT_K, t.glu, t.out, (__nv_bfloat16*)t.out_hi, (__nv_bfloat16*)t.out_lo, t.err};
    const int tiles = t.pairs / XT_N + (t.E < t.pairs ? t.E : t.pairs);      // an upper bound: every expert may end with a partial tile
    FT_REQUIRE(tiles <= 65535, "experts (tcgen05): %d pairs are too many", t.pairs);
    const dim3 grid(t.n_rows / XT_M, tiles);
    if (t.out) experts_tc_kernel<XT_ROWS><<<grid, XT_THREADS, XT_SMEM, stream>>>(mw, mh, ml, a);
    else if (t.act == FT_ACT_RELU2) experts_tc_kernel<XT_RELU2><<<grid, XT_THREADS, XT_SMEM, stream>>>(mw, mh, ml, a);
    else experts_tc_kernel<XT_GLU><<<grid, XT_THREADS, XT_SMEM, stream>>>(mw, mh, ml, a);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace ft
