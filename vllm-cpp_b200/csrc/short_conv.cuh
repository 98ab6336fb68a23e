// A short causal convolution over time, per channel, on a segment of a request's tokens held in registers:
//
//   y[t, c] = sum_j w[c, j] u[t - (J - 1) + j, c],     u = x + pre_bias,
//
// the J - 1 inputs before a step's first token read from the request's state slot (rows 0 .. J - 2, oldest first; zero at
// admission, which is "zeros before the start": the bias is never added to them) and the step's last J - 1 inputs left there.
// A thread owns VW neighbouring channels and a segment of SEG tokens; all its loads are issued before the first is used.
// J is at most MAXJ; taps are kept aligned to the window's end, absent ones are zero.  Segments are at least MAXJ - 1 tokens
// long, so only a request's first segment reads the state, and that thread alone rewrites it.
#pragma once
#include "common.cuh"

template <typename T, int VW> __device__ __forceinline__ void conv_load(const T* p, float (&v)[VW]) {
#pragma unroll
    for (int e = 0; e < VW; ++e) v[e] = to_f32<T>(p[e]);
}
template <> __device__ __forceinline__ void conv_load<__nv_bfloat16, 2>(const __nv_bfloat16* p, float (&v)[2]) {
    const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    v[0] = f.x;
    v[1] = f.y;
}
template <> __device__ __forceinline__ void conv_load<float, 2>(const float* p, float (&v)[2]) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x;
    v[1] = f.y;
}

// w: the taps of the thread's first channel ([VW][J] floats, contiguous) aligned to the end of a window of MAXJ.
template <int MAXJ, int VW>
__device__ __forceinline__ void conv_taps(const float* w, int J, int live, float (&taps)[MAXJ][VW]) {
#pragma unroll
    for (int m = 0; m < MAXJ; ++m)
#pragma unroll
        for (int e = 0; e < VW; ++e) {
            const int j = m - (MAXJ - J);
            taps[m][e] = (j >= 0 && e < live) ? w[e * J + j] : 0.0f;
        }
}

// h[i]: the input at token seg0 - (MAXJ - 1) + i of the request (x points at the request's first row and the thread's first
// channel; st at the slot's first row, rows `C` apart).  live: channels of the thread that exist.
template <typename T, int MAXJ, int SEG, int VW>
__device__ __forceinline__ void conv_window(const T* x, long long ldx, const float* st, int C, const float (&pb)[VW], int J, int seg0,
                                            int len, int live, float (&h)[MAXJ - 1 + SEG][VW]) {
#pragma unroll
    for (int i = 0; i < MAXJ - 1 + SEG; ++i) {
        const int li = seg0 - (MAXJ - 1) + i;
#pragma unroll
        for (int e = 0; e < VW; ++e) h[i][e] = 0.0f;
        if (i < MAXJ - J || li >= len) continue;
        if (li >= 0) {
            if (live == VW) {
                conv_load<T, VW>(x + (size_t)li * ldx, h[i]);
            } else {
                h[i][0] = to_f32<T>(x[(size_t)li * ldx]);
            }
#pragma unroll
            for (int e = 0; e < VW; ++e) h[i][e] += pb[e];
        } else {
#pragma unroll
            for (int e = 0; e < VW; ++e)
                if (e < live) h[i][e] = st[(size_t)(J - 1 + li) * C + e];
        }
    }
}

// The request's last J - 1 inputs into the slot, by the thread of its first segment after conv_window has read it.  Rows that
// stay move down; ascending rows never read what this loop has written.
template <typename T, int VW>
__device__ __forceinline__ void conv_keep(const T* x, long long ldx, float* st, int C, const float (&pb)[VW], int J, int len, int live) {
    for (int j = 0; j < J - 1; ++j) {
        const int li = len - (J - 1) + j;
#pragma unroll
        for (int e = 0; e < VW; ++e)
            if (e < live) st[(size_t)j * C + e] = li >= 0 ? to_f32<T>(x[(size_t)li * ldx + e]) + pb[e] : st[(size_t)(j + len) * C + e];
    }
}
