// Kernels that treat every coordinate by itself:
//
//   add_tanh_norm_kernel   the norm without statistics: x += mult * delta (+ mult2 * delta2: two
//                          mixers' results), out = tanh(alpha * x) * gain + shift.  The sum is written back to the float
//                          residual stream; nothing about a row needs the whole row, so a CTA takes any run of coordinates.
//   act_rows_kernel        the activation between the two matrices of a feed-forward without a gate: the square of relu, or
//                          gelu by its definition z Phi(z), Phi through erf.
//
// Arithmetic is float in both precisions.  The reference has RMS norms and gated feed-forwards only (src/kernels/layernorm.cu,
// src/kernels/activation.cu).
#include "common.cuh"

template <typename T, int V> struct PwVec;
template <typename T> struct PwVec<T, 1> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_f32<T>(*p); }
    static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { *p = from_f32<T>(v[0]); }
};
template <int V> struct PwVec<float, V> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[V]) {
#pragma unroll
        for (int i = 0; i < V; i += 4) {
            const float4 q = *reinterpret_cast<const float4*>(p + i);
            v[i] = q.x; v[i + 1] = q.y; v[i + 2] = q.z; v[i + 3] = q.w;
        }
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[V]) {
#pragma unroll
        for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    }
};
template <> struct PwVec<float, 1> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[1]) { v[0] = *p; }
    static __device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
};
template <> struct PwVec<__nv_bfloat16, 8> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[8]) {
        const uint4 q = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&q);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            v[2 * i] = f.x;
            v[2 * i + 1] = f.y;
        }
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[8]) {
        uint4 q;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&q);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = q;
    }
};

// ------------------------------------------------------------------------------------------- norm
// Grid-stride over vectors of V coordinates; the row and column of a vector advance with the stride.
template <typename T, int V>
__global__ void __launch_bounds__(256)
add_tanh_norm_kernel(float* __restrict__ residual, const T* __restrict__ delta, const T* __restrict__ delta2, const float* __restrict__ alpha,
                     const float* __restrict__ gain, const float* __restrict__ shift, T* __restrict__ out, const int* __restrict__ row_index,
                     int n_rows, int hidden, float mult, float mult2) {
    const int vpr = hidden / V;                          // vectors per row
    const float slope = *alpha;
    pdl_start();
    const long long total = (long long)n_rows * vpr;
    for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
        const int o = (int)(idx / vpr), c = (int)(idx - (long long)o * vpr) * V;
        const size_t row = row_index ? (size_t)row_index[o] : (size_t)o;
        float x[V], g[V], b[V];
        PwVec<float, V>::load(residual + row * hidden + c, x);
        PwVec<float, V>::load(gain + c, g);
        PwVec<float, V>::load(shift + c, b);
        if (delta) {
            float d[V];
            PwVec<T, V>::load(delta + row * hidden + c, d);
#pragma unroll
            for (int i = 0; i < V; ++i) x[i] = fmaf(mult, d[i], x[i]);
            if (delta2) {
                PwVec<T, V>::load(delta2 + row * hidden + c, d);
#pragma unroll
                for (int i = 0; i < V; ++i) x[i] = fmaf(mult2, d[i], x[i]);
            }
            if (!row_index) PwVec<float, V>::store(residual + row * hidden + c, x);
        }
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] = fmaf(tanhf(slope * x[i]), g[i], b[i]);
        PwVec<T, V>::store(out + (size_t)o * hidden + c, x);
    }
}

template <typename T, int V>
static int launch_tanh_norm(float* residual, const void* delta, const void* delta2, const float* alpha, const float* gain, const float* shift, void* out,
                            const int* row_index, int n_rows, int hidden, float mult, float mult2, cudaStream_t s) {
    const long long want = ((long long)n_rows * (hidden / V) + 255) / 256, cap = (long long)vcb_sm_count() * 16;
    vcb_launch(add_tanh_norm_kernel<T, V>, (int)(want < cap ? want : cap), 256, 0, s, residual, (const T*)delta, (const T*)delta2, alpha, gain,
               shift, (T*)out, row_index, n_rows, hidden, mult, mult2);
    return vcb_last_error();
}

// alpha: float [1].  row_index (may be null): output row o reads row row_index[o], and nothing is written back.
VCB_EXPORT int vcb_add_tanh_norm(float* residual, const void* delta, const void* delta2, const float* alpha, const float* gain, const float* shift,
                                 void* out, const int* row_index, int n_rows, int hidden, float mult, float mult2, int dtype, void* stream) {
    if (n_rows <= 0) return 0;
    if (!residual || (delta2 && !delta) || !alpha || !gain || !shift || !out || hidden <= 0) return VCB_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const bool aligned = !(((uintptr_t)residual | (uintptr_t)delta | (uintptr_t)delta2 | (uintptr_t)gain | (uintptr_t)shift | (uintptr_t)out) & 15);
    if (dtype == VCB_F32) {
        if (aligned && hidden % 4 == 0) return launch_tanh_norm<float, 4>(residual, delta, delta2, alpha, gain, shift, out, row_index, n_rows, hidden, mult, mult2, s);
        return launch_tanh_norm<float, 1>(residual, delta, delta2, alpha, gain, shift, out, row_index, n_rows, hidden, mult, mult2, s);
    }
    if (dtype != VCB_BF16) return VCB_ERR_BAD_ARG;
    if (aligned && hidden % 8 == 0) return launch_tanh_norm<__nv_bfloat16, 8>(residual, delta, delta2, alpha, gain, shift, out, row_index, n_rows, hidden, mult, mult2, s);
    return launch_tanh_norm<__nv_bfloat16, 1>(residual, delta, delta2, alpha, gain, shift, out, row_index, n_rows, hidden, mult, mult2, s);
}

// ------------------------------------------------------------------------------------- activations
enum { ACT_RELU_SQUARED = 0, ACT_GELU_ERF = 1 };

template <int ACT> __device__ __forceinline__ float pw_act(float z) {
    if (ACT == ACT_RELU_SQUARED) {
        const float r = fmaxf(z, 0.0f);
        return r * r;
    }
    return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f));
}

template <typename T, int V, int ACT>
__global__ void __launch_bounds__(256) act_rows_kernel(const T* x, T* out, long long n_vec) {
    pdl_start();
    for (long long v = (long long)blockIdx.x * blockDim.x + threadIdx.x; v < n_vec; v += (long long)gridDim.x * blockDim.x) {
        float f[V];
        PwVec<T, V>::load(x + v * V, f);
#pragma unroll
        for (int i = 0; i < V; ++i) f[i] = pw_act<ACT>(f[i]);
        PwVec<T, V>::store(out + v * V, f);
    }
}

template <typename T, int V>
static int launch_act(const void* x, void* out, long long n, int act, cudaStream_t s) {
    const long long n_vec = n / V, want = (n_vec + 255) / 256, cap = (long long)vcb_sm_count() * 16;
    const int blocks = (int)(want < cap ? want : cap);
    if (act == ACT_RELU_SQUARED) vcb_launch(act_rows_kernel<T, V, ACT_RELU_SQUARED>, blocks, 256, 0, s, (const T*)x, (T*)out, n_vec);
    else vcb_launch(act_rows_kernel<T, V, ACT_GELU_ERF>, blocks, 256, 0, s, (const T*)x, (T*)out, n_vec);
    return vcb_last_error();
}

// out = act(x) over n contiguous elements (out may be x).
VCB_EXPORT int vcb_act_rows(const void* x, void* out, long long n, int act, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (!x || !out || (act != ACT_RELU_SQUARED && act != ACT_GELU_ERF)) return VCB_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const bool aligned = !(((uintptr_t)x | (uintptr_t)out) & 15);
    if (dtype == VCB_F32) return aligned && n % 4 == 0 ? launch_act<float, 4>(x, out, n, act, s) : launch_act<float, 1>(x, out, n, act, s);
    if (dtype != VCB_BF16) return VCB_ERR_BAD_ARG;
    return aligned && n % 8 == 0 ? launch_act<__nv_bfloat16, 8>(x, out, n, act, s) : launch_act<__nv_bfloat16, 1>(x, out, n, act, s);
}
