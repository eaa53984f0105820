// The joint of the pre-norm layer form (FT_LAYER_PRENORM): the ONE kernel between two GEMM chains of a layer, one CTA per row.
// It gathers the sublayer's result (a projected row, optionally gated by one number per token, and / or the chosen experts'
// rows), scales it coordinate by coordinate, adds it to the stream, adds what comes ahead of a pass over looped layers, and
// norms the row for what reads it next, writing its bf16 planes as well.  A step's first joint fills the stream from the
// embedding tables instead.  Everything is fp32; the embedding tables are bf16.
#include "common.cuh"
#include "ft_internal.h"
#include "rows.cuh"

namespace ft {
namespace {

// V: columns per thread and pass (4 when the width is a multiple of four and every row starts on 16 bytes)
template <int V>
__device__ __forceinline__ void add_embedding(float (&x)[V], const PreNormArgs& a, int token, int pos, int c) {
    float e[V];
    ld_cols_bf16<V>(e, (const __nv_bfloat16*)a.embed + (size_t)token * a.W + c);
    if (a.pos_embed) {
        float p[V];
        ld_cols_bf16<V>(p, (const __nv_bfloat16*)a.pos_embed + (size_t)pos * a.W + c);
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] += fmaf(e[i], a.embed_scale, p[i]);
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] = fmaf(e[i], a.embed_scale, x[i]);
    }
}

template <int V>
__global__ void __launch_bounds__(256) prenorm_joint_kernel(PreNormArgs a) {
    __shared__ float red[33];
    extern __shared__ __align__(16) float row[];          // [W]: the new row of the stream
    const int t = blockIdx.x, W = a.W;
    const bool emb = a.first || a.re_embed;
    const int token = emb ? a.tokens[t] : 0, pos = emb ? a.positions[t] : 0;
    float g0 = 1.f;
    if (a.y_gate) g0 = 1.f / (1.f + expf(-a.y_gate[(size_t)t * a.ldg]));
    float* xr = a.x + (size_t)t * W;
    float total = 0.f;
    for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
        float x[V], v[V];
        if (a.first) {
#pragma unroll
            for (int i = 0; i < V; ++i) x[i] = 0.f;
            add_embedding<V>(x, a, token, pos, c);
        } else {
            float y[V];
#pragma unroll
            for (int i = 0; i < V; ++i) y[i] = 0.f;
            ld_cols<V>(x, xr + c);
            if (a.y0) {
                ld_cols<V>(v, a.y0 + (size_t)t * W + c);
#pragma unroll
                for (int i = 0; i < V; ++i) y[i] = g0 * v[i];
            }
            for (int k = 0; k < a.top; ++k) {
                ld_cols<V>(v, a.eout + (size_t)a.slot_pos[(size_t)t * a.top + k] * W + c);
                const float wk = a.wt[(size_t)t * a.top + k];
#pragma unroll
                for (int i = 0; i < V; ++i) y[i] = fmaf(wk, v[i], y[i]);
            }
            if (a.gain) {
                ld_cols<V>(v, a.gain + c);
#pragma unroll
                for (int i = 0; i < V; ++i) x[i] = fmaf(v[i], y[i], x[i]);
            } else {
#pragma unroll
                for (int i = 0; i < V; ++i) x[i] += y[i];
            }
            if (a.trail) st_cols<V>(a.trail + (size_t)t * W + c, x);
            if (a.re_embed) add_embedding<V>(x, a, token, pos, c);
        }
        if (a.pre_add) {
            ld_cols<V>(v, a.pre_add + c);
#pragma unroll
            for (int i = 0; i < V; ++i) x[i] += v[i];
        }
        st_cols<V>(xr + c, x);
        st_cols<V>(row + c, x);
#pragma unroll
        for (int i = 0; i < V; ++i) total = fmaf(x[i], x[i], total);
    }
    const float r = 1.f / sqrtf(cta_total(total, red) / (float)W + a.eps);
    __nv_bfloat16 *hi = (__nv_bfloat16*)a.hi, *lo = (__nv_bfloat16*)a.lo;
    for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
        float x[V], w[V];
        ld_cols<V>(x, row + c);
        ld_cols<V>(w, a.nw + c);
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] = x[i] * r * w[i];
        const size_t at = (size_t)t * W + c;
        st_cols<V>(a.hn + at, x);
        if (hi) st_planes<V>(hi + at, lo + at, x);
    }
}

}  // namespace

int launch_prenorm_joint(const PreNormArgs& a, int T, cudaStream_t stream) {
    FT_REQUIRE(a.x && a.hn && a.nw && (a.first || a.y0 || a.top > 0) && (!(a.first || a.re_embed) || (a.tokens && a.positions && a.embed)),
               "pre-norm joint: missing operands");
    const size_t smem = (size_t)a.W * 4;
    FT_REQUIRE(smem <= 160 * 1024, "pre-norm joint: width %d is too large", a.W);
    auto al = [](const void* p, size_t n) { return ((uintptr_t)p & (n - 1)) == 0; };
    const bool v4 = a.W % 4 == 0 && al(a.x, 16) && al(a.hn, 16) && al(a.y0, 16) && al(a.eout, 16) && al(a.gain, 16) && al(a.pre_add, 16) &&
                    al(a.nw, 16) && al(a.trail, 16) && al(a.embed, 8) && al(a.pos_embed, 8) && al(a.hi, 8) && al(a.lo, 8);
    if (smem > 48 * 1024) {
        static PerDeviceFlag attr;
        if (!attr.done()) {
            FT_CHECK_CUDA(cudaFuncSetAttribute(prenorm_joint_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
            FT_CHECK_CUDA(cudaFuncSetAttribute(prenorm_joint_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
            attr.mark();
        }
    }
    if (v4) prenorm_joint_kernel<4><<<T, 256, smem, stream>>>(a);
    else prenorm_joint_kernel<1><<<T, 256, smem, stream>>>(a);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace ft
