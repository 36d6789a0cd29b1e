// GELU for results that are rounded to bf16.
#pragma once
#include "common.cuh"

// erf to 1.5e-7 (Abramowitz & Stegun, Handbook of Mathematical Functions, 7.1.26)
__device__ __forceinline__ float gelu_bf16(float z) {
    const float x = fabsf(z) * 0.70710678f;
    const float t = __fdividef(1.0f, fmaf(0.3275911f, x, 1.0f));
    float p = fmaf(1.061405429f, t, -1.453152027f);
    p = fmaf(p, t, 1.421413741f);
    p = fmaf(p, t, -0.284496736f);
    p = fmaf(p, t, 0.254829592f);
    const float e = 1.0f - p * t * __expf(-x * x);
    return 0.5f * z * (1.0f + copysignf(e, z));
}
