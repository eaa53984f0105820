// Per-head projections on tcgen05: C[t, h, n] = sum_k A[t, h, k] * W[h][n, k] for the heads side by side in the columns of one
// buffer (queries folded into latent space, values expanded out of it).  Every head is a small product of its own (K one head's
// or one latent's size), so a launch covers all of them: CTA = (128 output features, NT tokens, head).
//
//   D[128 features x NT tokens] in TMEM = W tile (A operand, bf16) x token tile (B operand, the fp32 activations as bf16 hi + lo
//   planes: two products into one fp32 accumulator, about 16 mantissa bits of the activation).
//
// Both operands are K-major, 64 columns of K per block, rows of 128 bytes swizzled as the tensor core reads them.  256 threads
// bring the blocks in (W by asynchronous copies, activations through registers, one block ahead of the products), one thread
// issues the products; a block's buffer is free again when its products have been committed.  A lane of TMEM is a feature, so
// the epilogue writes 32 consecutive columns of C per warp and token, through the sigmoid gate when there is one.
#include "common.cuh"
#include "ft_internal.h"

#include <algorithm>

namespace ft {
namespace {

constexpr int HT_THREADS = 256, HT_ROWS = 128, HT_KB = 64, HT_SPIN = 1 << 20;

__device__ __forceinline__ bool ht_wait(uint64_t* bar, uint32_t parity) {
    for (int i = 0; i < HT_SPIN; ++i)
        if (mbar_try_wait(bar, parity)) return true;
    return false;
}
__device__ __forceinline__ void ht_copy16(uint32_t dst_smem, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst_smem), "l"(src) : "memory");
}

template <int NT>
__global__ void __launch_bounds__(HT_THREADS) linear_heads_kernel(LinearArgs a, int* err) {
    constexpr int W_BYTES = HT_ROWS * 128, X_BYTES = NT * 128, STAGE = W_BYTES + 2 * X_BYTES;
    constexpr int COLS = NT < 32 ? 32 : NT;
    constexpr int PIECES = (NT * 8 + HT_THREADS - 1) / HT_THREADS;      // (token row, 8 columns) pieces per thread and block
    extern __shared__ uint8_t ht_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ht_raw) + 1023) & ~uintptr_t(1023));
    __shared__ uint64_t freed[2];
    __shared__ uint32_t tmem_slot;
    __shared__ int dead;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int n0 = blockIdx.x * HT_ROWS, t0 = blockIdx.y * NT, p = blockIdx.z;
    const float* X = a.A + (size_t)p * a.a_col_stride;
    const __nv_bfloat16* W = a.W + (size_t)p * a.w_stride;
    if (tid == 0) {
        mbar_init(&freed[0], 1);
        mbar_init(&freed[1], 1);
        dead = 0;
        fence_mbar_init();
    }
    if (warp == 0) {
        tmem_alloc(&tmem_slot, COLS);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot, base = smem_u32(smem);
    const int nkb = (a.K + HT_KB - 1) / HT_KB;

    float4 xr[PIECES][2];
    auto load_x = [&](int kb) {
#pragma unroll
        for (int i = 0; i < PIECES; ++i) {
            const int idx = tid + i * HT_THREADS, r = idx >> 3, k = kb * HT_KB + (idx & 7) * 8;
            xr[i][0] = xr[i][1] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r < NT && t0 + r < a.M && k < a.K) {                    // K is a multiple of 8
                const float* src = X + (size_t)(t0 + r) * a.lda + k;
                xr[i][0] = *reinterpret_cast<const float4*>(src);
                xr[i][1] = *reinterpret_cast<const float4*>(src + 4);
            }
        }
    };
    auto load_w = [&](int kb, int buf) {
        for (int idx = tid; idx < HT_ROWS * 8; idx += HT_THREADS) {
            const int r = idx >> 3, ch = idx & 7, k = kb * HT_KB + ch * 8;
            const uint32_t off = buf * STAGE + r * 128 + ((ch ^ (r & 7)) << 4);
            if (n0 + r < a.N && k < a.K) ht_copy16(base + off, W + (size_t)(n0 + r) * a.ldw + k);
            else *reinterpret_cast<uint4*>(smem + off) = make_uint4(0u, 0u, 0u, 0u);
        }
    };
    load_x(0);
    bool ok = true;
    for (int kb = 0; kb < nkb; ++kb) {
        const int buf = kb & 1;
        if (kb >= 2) ok = ht_wait(&freed[buf], ((kb >> 1) - 1) & 1);
        if (!ok) dead = 1;
        load_w(kb, buf);
#pragma unroll
        for (int i = 0; i < PIECES; ++i) {
            const int idx = tid + i * HT_THREADS, r = idx >> 3, ch = idx & 7;
            if (r < NT) {
                const float v[8] = {xr[i][0].x, xr[i][0].y, xr[i][0].z, xr[i][0].w, xr[i][1].x, xr[i][1].y, xr[i][1].z, xr[i][1].w};
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    hi[e] = pack_bf16(v[2 * e], v[2 * e + 1]);
                    lo[e] = pack_bf16(v[2 * e] - bf16_lo(hi[e]), v[2 * e + 1] - bf16_hi(hi[e]));
                }
                uint8_t* dst = smem + buf * STAGE + W_BYTES + r * 128 + ((ch ^ (r & 7)) << 4);
                *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *reinterpret_cast<uint4*>(dst + X_BYTES) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
        }
        if (kb + 1 < nkb) load_x(kb + 1);
        asm volatile("cp.async.wait_all;" ::: "memory");
        fence_proxy_async();
        __syncthreads();
        if (dead) break;                                               // every thread sees the same value behind the barrier
        if (tid == 0) {
            const uint32_t idesc = umma_idesc_bf16(HT_ROWS, NT);
            const uint64_t wd = umma_desc_k128(base + buf * STAGE), xd = umma_desc_k128(base + buf * STAGE + W_BYTES),
                           ld = umma_desc_k128(base + buf * STAGE + W_BYTES + X_BYTES);
            const int steps = min(4, (a.K - kb * HT_KB + 15) / 16);
            for (int k = 0; k < steps; ++k) {
                umma_bf16(tmem, wd + 2 * k, xd + 2 * k, idesc, (kb | k) != 0);
                umma_bf16(tmem, wd + 2 * k, ld + 2 * k, idesc, 1);
            }
            umma_commit(&freed[buf]);
        }
    }
    // the last block's commit covers every product before it
    if (!dead) {
        ok = ht_wait(&freed[(nkb - 1) & 1], ((nkb - 1) >> 1) & 1);
        tc_fence_after();
        __syncwarp();
        if (ok) {
            const int f = n0 + (warp & 3) * 32 + lane;
            const uint32_t lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
            for (int c = (warp >> 2) * 16; c < NT; c += 32) {
                if (t0 + c >= a.M) break;                              // uniform
                const int nt = min(16, a.M - t0 - c);
                const size_t col = (size_t)p * a.c_col_stride + f;
                float v[16], g[16];
                if (a.gate && f < a.N) {                               // all of them on the way before the first is used
                    const float* gp = a.gate + (size_t)(t0 + c) * a.ldg + col;
#pragma unroll
                    for (int i = 0; i < 16; ++i) g[i] = i < nt ? gp[(size_t)i * a.ldg] : 0.f;
                }
                __syncwarp();
                tmem_ld16(lanes + c, v);
                if (f < a.N) {
                    if (a.gate) {
#pragma unroll
                        for (int i = 0; i < 16; ++i) v[i] *= 1.f / (1.f + expf(-g[i]));
                    }
                    const size_t at = (size_t)(t0 + c) * a.ldc + col;
                    if (a.C16) {
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (i < nt) a.C16[at + (size_t)i * a.ldc] = __float2bfloat16_rn(v[i] * a.c16_scale);
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (i < nt) a.C[at + (size_t)i * a.ldc] = v[i];
                    }
                }
                __syncwarp();
            }
        } else {
            dead = 1;
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        tc_fence_after();
        tmem_dealloc(tmem, COLS);
    }
    if (tid == 0 && dead && err) *err = 1;
}

template <int NT>
int launch_nt(const LinearArgs& a, int* err, cudaStream_t stream) {
    constexpr int SMEM = 1024 + 2 * (HT_ROWS * 128 + 2 * NT * 128);
    static PerDeviceFlag attr;
    if (!attr.done()) {
        FT_CHECK_CUDA(cudaFuncSetAttribute(linear_heads_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM));
        attr.mark();
    }
    const dim3 grid((a.N + HT_ROWS - 1) / HT_ROWS, (a.M + NT - 1) / NT, a.P);
    linear_heads_kernel<NT><<<grid, HT_THREADS, SMEM, stream>>>(a, err);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace

bool linear_heads_ok(const LinearArgs& a) {
    return !a.seg && !a.a_rows && a.epi == LIN_PLAIN && a.K % 32 == 0 && a.N % 32 == 0 && a.K >= 32 && a.lda % 4 == 0 && a.ldw % 8 == 0 &&
           a.a_col_stride % 4 == 0 && a.w_stride % 8 == 0 && ((uintptr_t)a.A & 15) == 0 && ((uintptr_t)a.W & 15) == 0 && a.P <= 65535 &&
           (a.M + 15) / 16 <= 65535;
}

int launch_linear_heads(const LinearArgs& a, int* err, cudaStream_t stream) {
    FT_REQUIRE(linear_heads_ok(a), "per-head projections (tcgen05): sizes or alignment do not fit");
    if (a.M <= 0) return 0;
    if (a.M <= 16) return launch_nt<16>(a, err, stream);
    if (a.M <= 32) return launch_nt<32>(a, err, stream);
    if (a.M <= 64) return launch_nt<64>(a, err, stream);
    return launch_nt<128>(a, err, stream);
}

}  // namespace ft
