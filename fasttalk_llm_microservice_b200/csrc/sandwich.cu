// The joint of the sandwich layer form (FT_LAYER_SANDWICH): the ONE kernel between two GEMM chains of a layer, one CTA per row.
// It gathers the sublayer's result (the scaled sum of up to two branch results, or the experts' rows plus a dense or shared
// result and its bias), norms it, adds it to the stream, and norms the stream for what reads it next, writing the bf16 planes as
// well — or, ahead of a pass over looped layers, lays the stream down beside the embedding output.  A step's first joint
// fills the stream from the embedding table.  Everything is fp32; the embedding table is bf16.
#include "common.cuh"
#include "ft_internal.h"
#include "rows.cuh"

namespace ft {
namespace {

// V: columns per thread and pass (4 when the width is a multiple of four and every row starts on 16 bytes)
template <int V>
__device__ __forceinline__ void put_row(float* f32, void* hi, void* lo, size_t at, const float (&v)[V]) {
    st_cols<V>(f32 + at, v);
    if (hi) st_planes<V>((__nv_bfloat16*)hi + at, (__nv_bfloat16*)lo + at, v);
}

template <int V>
__global__ void __launch_bounds__(256) sandwich_joint_kernel(SandwichArgs a) {
    __shared__ float red[33];
    extern __shared__ __align__(16) float row[];          // [W]: the sublayer's result, then the new row of the stream
    const int t = blockIdx.x, W = a.W;
    const bool sub = a.y0 || a.y1 || a.top > 0;
    float* xr = a.x + (size_t)t * W;
    float r1 = 0.f;
    if (sub) {
        float ss = 0.f;
        for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
            float y[V], v[V];
#pragma unroll
            for (int i = 0; i < V; ++i) y[i] = 0.f;
            for (int k = 0; k < a.top; ++k) {
                ld_cols<V>(v, a.eout + (size_t)a.slot_pos[(size_t)t * a.top + k] * W + c);
                const float wk = a.wt[(size_t)t * a.top + k];
#pragma unroll
                for (int i = 0; i < V; ++i) y[i] = fmaf(wk, v[i], y[i]);
            }
            if (a.y0) {
                ld_cols<V>(v, a.y0 + (size_t)t * W + c);
#pragma unroll
                for (int i = 0; i < V; ++i) y[i] = fmaf(a.s0, v[i], y[i]);
            }
            if (a.b0) {
                ld_cols<V>(v, a.b0 + c);
#pragma unroll
                for (int i = 0; i < V; ++i) y[i] += v[i];
            }
            if (a.y1) {
                ld_cols<V>(v, a.y1 + (size_t)t * W + c);
#pragma unroll
                for (int i = 0; i < V; ++i) y[i] = fmaf(a.s1, v[i], y[i]);
            }
            st_cols<V>(row + c, y);
#pragma unroll
            for (int i = 0; i < V; ++i) ss = fmaf(y[i], y[i], ss);
        }
        r1 = 1.f / sqrtf(cta_total(ss, red) / (float)W + a.eps);
    }
    const __nv_bfloat16* emb = a.tokens ? (const __nv_bfloat16*)a.embed + (size_t)a.tokens[t] * W : nullptr;
    float s2 = 0.f;
    for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
        float x[V];
        if (emb) {
            ld_cols_bf16<V>(x, emb + c);
#pragma unroll
            for (int i = 0; i < V; ++i) x[i] *= a.embed_scale;
        } else {
            ld_cols<V>(x, xr + c);
        }
        if (sub) {
            float y[V], w[V];
            ld_cols<V>(y, row + c);
            ld_cols<V>(w, a.post_w + c);
#pragma unroll
            for (int i = 0; i < V; ++i) x[i] += y[i] * r1 * w[i];
        }
        if (sub || emb) st_cols<V>(xr + c, x);
        if (a.cat_x) put_row<V>(a.cat, a.cat_hi, a.cat_lo, (size_t)t * 2 * W + c, x);
        if (a.cat_x0) put_row<V>(a.cat, a.cat_hi, a.cat_lo, (size_t)t * 2 * W + W + c, x);
        st_cols<V>(row + c, x);
#pragma unroll
        for (int i = 0; i < V; ++i) s2 = fmaf(x[i], x[i], s2);
    }
    if (!a.next_w) return;
    const float r2 = 1.f / sqrtf(cta_total(s2, red) / (float)W + a.eps);
    for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
        float x[V], w[V];
        ld_cols<V>(x, row + c);
        ld_cols<V>(w, a.next_w + c);
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] = x[i] * r2 * w[i];
        put_row<V>(a.hn, a.hi, a.lo, (size_t)t * W + c, x);
    }
}

}  // namespace

int launch_sandwich_joint(const SandwichArgs& a, int T, cudaStream_t stream) {
    const bool sub = a.y0 || a.y1 || a.top > 0;
    FT_REQUIRE(a.x && (!sub || a.post_w) && (!a.next_w || a.hn) && (a.next_w || a.cat_x) && (!(a.cat_x || a.cat_x0) || a.cat) &&
                   (!a.tokens || a.embed) && (!a.cat_x0 || a.tokens) && (a.top == 0 || (a.eout && a.wt && a.slot_pos)),
               "sandwich joint: missing operands");
    const size_t smem = (size_t)a.W * 4;
    FT_REQUIRE(smem <= 160 * 1024, "sandwich joint: width %d is too large", a.W);
    auto al = [](const void* p, size_t n) { return ((uintptr_t)p & (n - 1)) == 0; };
    const bool v4 = a.W % 4 == 0 && al(a.x, 16) && al(a.hn, 16) && al(a.y0, 16) && al(a.y1, 16) && al(a.b0, 16) && al(a.eout, 16) &&
                    al(a.post_w, 16) && al(a.next_w, 16) && al(a.cat, 16) && al(a.embed, 8) && al(a.hi, 8) && al(a.lo, 8) && al(a.cat_hi, 8) &&
                    al(a.cat_lo, 8);
    if (smem > 48 * 1024) {
        static PerDeviceFlag attr;
        if (!attr.done()) {
            FT_CHECK_CUDA(cudaFuncSetAttribute(sandwich_joint_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
            FT_CHECK_CUDA(cudaFuncSetAttribute(sandwich_joint_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
            attr.mark();
        }
    }
    if (v4) sandwich_joint_kernel<4><<<T, 256, smem, stream>>>(a);
    else sandwich_joint_kernel<1><<<T, 256, smem, stream>>>(a);
    FT_CHECK_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace ft
