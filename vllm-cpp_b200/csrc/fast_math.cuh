// Short forms of the functions that recurrences evaluate per element, on the special-function unit's ex2 and rcp (each good to
// about 2^-22 relative), and packed arithmetic on two floats at a time.
#pragma once
#include "common.cuh"

#define FM_LOG2E 1.4426950408889634f

__device__ __forceinline__ float fm_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float fm_rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// e^-z overflows to infinity for very negative z, whose reciprocal is the limit 0
__device__ __forceinline__ float fm_sigmoid(float z) { return fm_rcp(1.0f + fm_ex2(-FM_LOG2E * z)); }
__device__ __forceinline__ float fm_silu(float z) { return z * fm_sigmoid(z); }
// softplus(z) = max(z, 0) + log(1 + e), e = exp(-|z|).  log(1 + e) = 2 artanh(s) with s = e / (2 + e), at most 1/3, by the series
// of artanh, which keeps its relative accuracy where e is small (1 + e would lose it).
__device__ __forceinline__ float fm_softplus(float z) {
    const float e = fm_ex2(-FM_LOG2E * fabsf(z)), s = e * fm_rcp(2.0f + e), q = s * s;
    float p = 1.0f / 15.0f;
    p = fmaf(p, q, 1.0f / 13.0f);
    p = fmaf(p, q, 1.0f / 11.0f);
    p = fmaf(p, q, 1.0f / 9.0f);
    p = fmaf(p, q, 1.0f / 7.0f);
    p = fmaf(p, q, 1.0f / 5.0f);
    p = fmaf(p, q, 1.0f / 3.0f);
    p = fmaf(p, q, 1.0f);
    return fmaxf(z, 0.0f) + 2.0f * s * p;
}

typedef unsigned long long f32x2;      // two floats in a register pair
__device__ __forceinline__ f32x2 pack2f(float a, float b) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void unpack2f(f32x2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ float sum2f(f32x2 v) {
    float a, b;
    unpack2f(v, a, b);
    return a + b;
}
__device__ __forceinline__ f32x2 fma2f(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 mul2f(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
