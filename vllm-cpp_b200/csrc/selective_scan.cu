// A selective state space: per channel c a state of N numbers that decays and is driven by the token, with step sizes,
// drive and read-out made from the token itself,
//
//   s_n <- e^(dt a_n) s_n + (dt x) b_n  for n < N,     y = b'.s + d x  with read-out weights b' of the token,     out = silu(z) y
//
// (the channel's own a and d; b and b' are the same for all channels of a token: B and C below; dt = softplus(dt_pre + dt_bias)).
// x, dt_pre, B, C and z are rows of the activations' type; step sizes, exponentials, state,
// sums and the gate are float.  The state lives in the request's slot ([slots][I][N]), is read at the start of a request's
// portion and left there at its end.
//
//   selective_step_kernel    single tokens: a thread per channel and NPT states
//   selective_scan_kernel    portions: the same threads walk the request's tokens, whose step sizes, drives, B and C are made
//                            once per chunk in shared memory while the values of the chunk after are on their way
//
// Exponentials are ex2.approx (2^-22 relative) of dt * A log2(e); softplus and the gate are those of fast_math.cuh.  The reference has no recurrent mixer.
#include "fast_math.cuh"

struct SelectiveArgs {
    const void* x;              // [n, I] rows of T
    const void* dt_pre;         // [n, I]
    const void* b;              // [n, N]
    const void* c;              // [n, N]
    const void* z;              // [n, I]
    long long ldx, lddt, ldb, ldc, ldz;
    const float* dt_bias;       // [I]
    const float* a2;            // [I, N]: A * log2(e), A < 0
    const float* d;             // [I]
    float* state;               // [slots][I][N]
    void* out;                  // [n, I] of T
    long long ldo;
    const int* q_start;
    const int* state_slots;
    int I, N;
};

// NPT consecutive floats of a row of N (those beyond N: zero); quads where the row allows.
template <int NPT>
__device__ __forceinline__ void ss_load(const float* p, int n0, int N, bool quads, float (&v)[NPT]) {
    if (NPT >= 4 && quads && n0 + NPT <= N) {
#pragma unroll
        for (int i = 0; i + 3 < NPT; i += 4) {
            const float4 q = *reinterpret_cast<const float4*>(p + n0 + i);
            v[i] = q.x; v[i + 1] = q.y; v[i + 2] = q.z; v[i + 3] = q.w;
        }
        return;
    }
#pragma unroll
    for (int i = 0; i < NPT; ++i) v[i] = n0 + i < N ? p[n0 + i] : 0.0f;
}
template <int NPT>
__device__ __forceinline__ void ss_store(float* p, int n0, int N, bool quads, const float (&v)[NPT]) {
    if (NPT >= 4 && quads && n0 + NPT <= N) {
#pragma unroll
        for (int i = 0; i + 3 < NPT; i += 4) *reinterpret_cast<float4*>(p + n0 + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
        return;
    }
#pragma unroll
    for (int i = 0; i < NPT; ++i)
        if (n0 + i < N) p[n0 + i] = v[i];
}

// Grid (tiles of channels, requests); L lanes of a warp share a channel.
template <typename T, int NPT>
__global__ void __launch_bounds__(128) selective_step_kernel(SelectiveArgs a, int L) {
    const int per = 128 / L, ch = blockIdx.x * per + threadIdx.x / L, part = threadIdx.x % L;
    const bool there = ch < a.I;
    const int c = there ? ch : a.I - 1, n0 = part * NPT;
    const bool quads = (a.N & 3) == 0;
    float A[NPT];
    ss_load<NPT>(a.a2 + (size_t)c * a.N, n0, a.N, quads, A);
    const float bias = a.dt_bias[c], dc = a.d[c];
    const int r = blockIdx.y;
    const size_t row = (size_t)a.q_start[r];                 // the step's index arrays are older than the kernel before
    float* st = a.state + ((size_t)a.state_slots[r] * a.I + c) * a.N;
    pdl_start();
    float S[NPT];
    ss_load<NPT>(st, n0, a.N, quads, S);
    const float x = to_f32<T>(((const T*)a.x)[row * a.ldx + c]);
    const float dt = fm_softplus(to_f32<T>(((const T*)a.dt_pre)[row * a.lddt + c]) + bias);
    const float z = to_f32<T>(((const T*)a.z)[row * a.ldz + c]);
    const T* bp = (const T*)a.b + row * a.ldb;
    const T* cp = (const T*)a.c + row * a.ldc;
    const float dx = dt * x;
    float y = 0.0f;
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
        const bool in = n0 + i < a.N;
        const float bn = in ? to_f32<T>(bp[n0 + i]) : 0.0f, cn = in ? to_f32<T>(cp[n0 + i]) : 0.0f;
        S[i] = fmaf(fm_ex2(dt * A[i]), S[i], dx * bn);
        y = fmaf(S[i], cn, y);
    }
    for (int o = 1; o < L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (!there) return;
    ss_store<NPT>(st, n0, a.N, quads, S);
    if (part == 0) ((T*)a.out)[row * a.ldo + c] = from_f32<T>(fmaf(dc, x, y) * fm_silu(z));
}

// v[k], k = 0 .. L - 1: every lane's share of the sum of token k over the L lanes of a channel.  Returns, in lane `part`, the
// whole sum of token `part`: each round a lane keeps the half of its tokens that matches its bit and hands over the other.
template <int L>
__device__ __forceinline__ float ss_deal_sums(float (&v)[L], int part) {
#pragma unroll
    for (int half = L / 2; half > 0; half >>= 1) {
        const bool upper = part & half;
#pragma unroll
        for (int k = 0; k < half; ++k) {
            const float keep = upper ? v[k + half] : v[k], give = upper ? v[k] : v[k + half];
            v[k] = keep + __shfl_xor_sync(0xffffffffu, give, half);
        }
    }
    return v[0];
}

// Grid (tiles of CB channels, requests), CB * L threads; chunks of TC tokens.  Tokens beyond the portion's end are staged as
// dt = 0 and dx = 0, which leave the state as it is, so a chunk is always walked whole.  L tokens are walked together: their
// read-outs are independent of one another, and their sums over a channel's lanes are dealt out one token to a lane.
template <typename T, int NPT, int L, int CB, int TC>
__global__ void __launch_bounds__(CB * L) selective_scan_kernel(SelectiveArgs a) {
    constexpr int THREADS = CB * L, PER = (TC * CB + THREADS - 1) / THREADS, NP = L * NPT, PERN = (TC * NP + THREADS - 1) / THREADS;
    constexpr int GROUP = (L <= TC) ? L : 1;                  // tokens walked together
    static_assert(THREADS % NP == 0 && (TC % L == 0 || L > TC) && TC % (THREADS / NP) == 0, "whole rounds of staging");
    __shared__ __align__(16) float2 dts[TC][CB];              // dt, dt * x
    __shared__ __align__(16) float bs[TC][NP], cs[TC][NP];
    __shared__ float ys[TC][CB + 1];
    const int tid = threadIdx.x, part = tid % L, cl = tid / L, c0 = blockIdx.x * CB;
    const int c = min(c0 + cl, a.I - 1), n0 = part * NPT;
    const bool there = c0 + cl < a.I, quads = (a.N & 3) == 0;
    float S[NPT];
    f32x2 A2[NPT / 2], S2[NPT / 2];
    ss_load<NPT>(a.a2 + (size_t)c * a.N, n0, a.N, quads, S);
#pragma unroll
    for (int i = 0; i < NPT / 2; ++i) A2[i] = pack2f(S[2 * i], S[2 * i + 1]);
    const int sc = tid % CB, st0 = tid / CB;                  // staging: channel sc, tokens st0, st0 + L, ...
    const int scc = min(c0 + sc, a.I - 1);
    const float bias = a.dt_bias[scc], dc = a.d[scc];
    pdl_start();
    const int r = blockIdx.y;
    const int row0 = a.q_start[r], len = a.q_start[r + 1] - row0;
    if (len <= 0) return;
    float* st = a.state + ((size_t)a.state_slots[r] * a.I + c) * a.N;
    ss_load<NPT>(st, n0, a.N, quads, S);
#pragma unroll
    for (int i = 0; i < NPT / 2; ++i) S2[i] = pack2f(S[2 * i], S[2 * i + 1]);
    // every thread's own pointers to the values it stages next; a chunk advances them
    const T* xp = (const T*)a.x + (size_t)(row0 + st0) * a.ldx + scc;
    const T* dp = (const T*)a.dt_pre + (size_t)(row0 + st0) * a.lddt + scc;
    const T* zp = (const T*)a.z + (size_t)(row0 + st0) * a.ldz + scc;
    T* op = (T*)a.out + (size_t)(row0 + st0) * a.ldo + scc;
    const int nb = min(tid % NP, a.N - 1), tb = tid / NP;        // B and C: state nb, tokens tb, tb + THREADS / NP, ...
    const bool in = tid % NP < a.N;
    constexpr int TB = THREADS / NP;
    const T* bp = (const T*)a.b + (size_t)(row0 + tb) * a.ldb + nb;
    const T* cp = (const T*)a.c + (size_t)(row0 + tb) * a.ldc + nb;
    constexpr int ROWS = L < TC ? L : TC;                        // token rows the staging threads cover at once
    const long long sx = (long long)ROWS * a.ldx, sd = (long long)ROWS * a.lddt, sz = (long long)ROWS * a.ldz, so = (long long)ROWS * a.ldo,
                    sb = (long long)TB * a.ldb, scs = (long long)TB * a.ldc;
    T px[PER], pd[PER], pz[PER], pb[PERN], pc[PERN];          // a chunk's values on their way, as they are stored
#pragma unroll
    for (int k = 0; k < PER; ++k) px[k] = pd[k] = pz[k] = from_f32<T>(0.0f);
#pragma unroll
    for (int k = 0; k < PERN; ++k) pb[k] = pc[k] = from_f32<T>(0.0f);
    auto fetch = [&](int left) {                              // left: tokens from the chunk's first one on
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            if (st0 + k * L < min(left, TC)) {
                px[k] = *xp;
                pd[k] = *dp;
                pz[k] = *zp;
            }
            xp += sx;
            dp += sd;
            zp += sz;
        }
#pragma unroll
        for (int k = 0; k < PERN; ++k) {
            if (tb + k * TB < min(left, TC)) {
                pb[k] = *bp;
                pc[k] = *cp;
            }
            bp += sb;
            cp += scs;
        }
    };
    fetch(len);
    for (int t0 = 0; t0 < len; t0 += TC) {
        const int tc = min(TC, len - t0);
        float zk[PER], xk[PER];
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int t = st0 + k * L;
            xk[k] = to_f32<T>(px[k]);
            zk[k] = to_f32<T>(pz[k]);
            if (t < TC) {
                const float dt = t < tc ? fm_softplus(to_f32<T>(pd[k]) + bias) : 0.0f;
                dts[t][sc] = make_float2(dt, dt * xk[k]);
            }
        }
#pragma unroll
        for (int k = 0; k < PERN; ++k) {
            const int t = tb + k * TB;
            if (t < TC) {
                bs[t][tid % NP] = in ? to_f32<T>(pb[k]) : 0.0f;
                cs[t][tid % NP] = in ? to_f32<T>(pc[k]) : 0.0f;
            }
        }
        __syncthreads();
        if (t0 + TC < len) fetch(len - t0 - TC);
#pragma unroll
        for (int g = 0; g < TC; g += GROUP) {
            float y[GROUP];
#pragma unroll
            for (int k = 0; k < GROUP; ++k) {
                const float2 d = dts[g + k][cl];
                const f32x2 dt2 = pack2f(d.x, d.x), dx2 = pack2f(d.y, d.y);
                f32x2 y2 = pack2f(0.0f, 0.0f);
#pragma unroll
                for (int i = 0; i < NPT / 2; ++i) {
                    const float2 b2 = *reinterpret_cast<const float2*>(&bs[g + k][n0 + 2 * i]), c2 = *reinterpret_cast<const float2*>(&cs[g + k][n0 + 2 * i]);
                    float e0, e1;
                    unpack2f(mul2f(dt2, A2[i]), e0, e1);
                    S2[i] = fma2f(pack2f(fm_ex2(e0), fm_ex2(e1)), S2[i], mul2f(dx2, pack2f(b2.x, b2.y)));
                    y2 = fma2f(S2[i], pack2f(c2.x, c2.y), y2);
                }
                float u, v;
                unpack2f(y2, u, v);
                y[k] = u + v;
            }
            if constexpr (GROUP == L) {
                ys[g + part][cl] = ss_deal_sums<L>(y, part);
            } else {
                float v = y[0];
#pragma unroll
                for (int o = 1; o < L; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
                if (part == 0) ys[g][cl] = v;
            }
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int t = st0 + k * L;
            if (t < tc && c0 + sc < a.I) *op = from_f32<T>(fmaf(dc, xk[k], ys[t][sc]) * fm_silu(zk[k]));
            op += so;
        }
        // ys is written again only after the next chunk's first barrier
    }
#pragma unroll
    for (int i = 0; i < NPT / 2; ++i) unpack2f(S2[i], S[2 * i], S[2 * i + 1]);
    if (there) ss_store<NPT>(st, n0, a.N, quads, S);
}

template <typename T, int NPT, int L, int CB>
static void launch_scan(const SelectiveArgs& a, int n_reqs, cudaStream_t s) {
    vcb_launch(selective_scan_kernel<T, NPT, L, CB, (NPT > 4 ? 4 : 16)>, dim3((a.I + CB - 1) / CB, n_reqs), CB * L, 0, s, a);
}

template <typename T>
static int launch_selective(const SelectiveArgs& a, int n_reqs, int max_q_len, cudaStream_t s) {
    const int npt = a.N <= 128 ? 4 : 16;
    int L = 1;
    while (L * npt < a.N) L <<= 1;
    if (L > 32) return VCB_ERR_UNSUPPORTED;
    if (max_q_len == 1) {
        dim3 grid((a.I + 128 / L - 1) / (128 / L), n_reqs);
        if (npt == 4) vcb_launch(selective_step_kernel<T, 4>, grid, 128, 0, s, a, L);
        else vcb_launch(selective_step_kernel<T, 16>, grid, 128, 0, s, a, L);
        return vcb_last_error();
    }
    if (npt == 16) {
        if (L == 16) launch_scan<T, 16, 16, 16>(a, n_reqs, s);
        else launch_scan<T, 16, 32, 16>(a, n_reqs, s);
        return vcb_last_error();
    }
    // two states a thread where the channels alone leave the SMs with few warps
    if (a.N <= 32 && a.N > 1) {
        if (a.N <= 2) launch_scan<T, 2, 1, 32>(a, n_reqs, s);
        else if (a.N <= 4) launch_scan<T, 2, 2, 32>(a, n_reqs, s);
        else if (a.N <= 8) launch_scan<T, 2, 4, 32>(a, n_reqs, s);
        else if (a.N <= 16) launch_scan<T, 2, 8, 16>(a, n_reqs, s);
        else launch_scan<T, 2, 16, 8>(a, n_reqs, s);
        return vcb_last_error();
    }
    switch (L) {
        case 1: launch_scan<T, 4, 1, 32>(a, n_reqs, s); break;
        case 16: launch_scan<T, 4, 16, 8>(a, n_reqs, s); break;
        default: launch_scan<T, 4, 32, 8>(a, n_reqs, s); break;
    }
    return vcb_last_error();
}

VCB_EXPORT int vcb_selective_scan(const void* x, long long ldx, const void* dt_pre, long long lddt, const void* b, long long ldb,
                                  const void* c, long long ldc, const void* z, long long ldz, const float* dt_bias, const float* a2,
                                  const float* d, float* state, void* out, long long ldo, const int* q_start, const int* state_slots,
                                  int n_reqs, int max_q_len, int I, int N, int dtype, void* stream) {
    if (n_reqs <= 0 || max_q_len <= 0) return 0;
    if (!x || !dt_pre || !b || !c || !z || !dt_bias || !a2 || !d || !state || !out || I <= 0 || N <= 0 || n_reqs > 65535) return VCB_ERR_BAD_ARG;
    SelectiveArgs a{x, dt_pre, b, c, z, ldx, lddt, ldb, ldc, ldz, dt_bias, a2, d, state, out, ldo, q_start, state_slots, I, N};
    if (dtype == VCB_F32) return launch_selective<float>(a, n_reqs, max_q_len, (cudaStream_t)stream);
    if (dtype == VCB_BF16) return launch_selective<__nv_bfloat16>(a, n_reqs, max_q_len, (cudaStream_t)stream);
    return VCB_ERR_BAD_ARG;
}
