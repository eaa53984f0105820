// What the one-CTA-per-row kernels share: a sum over the CTA, and V consecutive fp32 or bf16 columns of a row at once.
#pragma once
#include "common.cuh"

namespace ft {

__device__ __forceinline__ float cta_total(float v, float* red) {      // red: >= 33 floats of shared memory
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

// V consecutive columns of a row at once: 16-byte loads and stores of fp32 (8-byte ones of bf16) when V == 4.
template <int V>
__device__ __forceinline__ void ld_cols(float (&d)[V], const float* p) {
    if constexpr (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        d[0] = t.x; d[1] = t.y; d[2] = t.z; d[3] = t.w;
    } else {
        d[0] = *p;
    }
}
template <int V>
__device__ __forceinline__ void st_cols(float* p, const float (&d)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(d[0], d[1], d[2], d[3]);
    else *p = d[0];
}
template <int V>
__device__ __forceinline__ void ld_cols_bf16(float (&d)[V], const __nv_bfloat16* p) {
    if constexpr (V == 4) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&t.x), b = *reinterpret_cast<const __nv_bfloat162*>(&t.y);
        d[0] = __low2float(a); d[1] = __high2float(a); d[2] = __low2float(b); d[3] = __high2float(b);
    } else {
        d[0] = __bfloat162float(*p);
    }
}
template <int V>
__device__ __forceinline__ void st_planes(__nv_bfloat16* hi, __nv_bfloat16* lo, const float (&d)[V]) {
    __nv_bfloat16 h[V], l[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
        h[i] = __float2bfloat16_rn(d[i]);
        l[i] = __float2bfloat16_rn(d[i] - __bfloat162float(h[i]));
    }
    if constexpr (V == 4) {
        *reinterpret_cast<uint2*>(hi) = *reinterpret_cast<const uint2*>(h);
        *reinterpret_cast<uint2*>(lo) = *reinterpret_cast<const uint2*>(l);
    } else {
        *hi = h[0];
        *lo = l[0];
    }
}

}  // namespace ft
