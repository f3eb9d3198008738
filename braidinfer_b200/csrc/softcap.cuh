// Capped attention scores: cap * tanh(score / cap), float32.
//
// tanh is used in two forms.  For |y| <= SOFTCAP_SMALL it is y P(y^2), P a polynomial of degree 5 that interpolates
// tanh(y) / y at the Chebyshev nodes of [0, SOFTCAP_SMALL^2] (relative error 3e-8 before rounding, 2e-7 in float32): plain
// multiply-adds, where the special-function pipe would be the attention kernels' bound.  Beyond, tanh(y) = 1 - 2 / (1 + exp(2y))
// (absolute error a few 1e-7).  A warp takes the first form for a tile of scores when every lane's scores allow it: scores
// rarely come near the cap.
#pragma once
#include "common.cuh"

#define SOFTCAP_SMALL 0.75f
__device__ __forceinline__ float tanh_small(float y) {
    const float z = y * y;
    float p = -0.0047115223f;
    p = fmaf(p, z, 0.019576216f);
    p = fmaf(p, z, -0.053341117f);
    p = fmaf(p, z, 0.1332534f);
    p = fmaf(p, z, -0.33332953f);
    return fmaf(y * z, p, y);
}
__device__ __forceinline__ float tanh_any(float y) {
    return 1.f - __fdividef(2.f, 1.f + exp2f(2.8853900817779268f * y));
}

// s[i] <- cap * tanh(s[i] * factor) for N scores a lane; the whole warp calls.
template <int N>
__device__ __forceinline__ void softcap_scores(float* s, float factor, float cap) {
    float top = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) top = fmaxf(top, fabsf(s[i]));
    if (__any_sync(0xffffffffu, !(top * fabsf(factor) <= SOFTCAP_SMALL))) {
#pragma unroll
        for (int i = 0; i < N; ++i) s[i] = cap * tanh_any(s[i] * factor);
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) s[i] = cap * tanh_small(s[i] * factor);
    }
}
