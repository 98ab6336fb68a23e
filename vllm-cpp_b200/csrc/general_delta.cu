// A generalised delta rule per head on a matrix S of key channels by value channels: the token decays S per key channel,
// removes, at a rate per key channel, what S held under the token's unit key, and adds the outer product of the plain key and
// the value; both terms read the old S:
//
//   u = k / sqrt(sum k^2 + eps),   w = exp(-rate * sigmoid(z + z_bias)),   a = sigmoid(a_pre + a_bias)
//   S <- diag(w) S - (a * u) (u^T S) + k v^T,     o = S^T r
//
// r, k, v, z and a_pre are rows of the activations' type; everything from there to o is float.  The state lives in the request's
// slot ([slots][H][dk][dv]), is read at the start of a request's portion and left there at its end.  With |k| = kn, k = kn u,
// and both sums over key channels that a token needs come from the old S:
//   p = u . S[:, c],  R = r . (w * S[:, c]);   S[:, c] = w * S[:, c] + u * (kn v_c - a p);   o_c = R - (r . (a u)) p + (r . k) v_c
// so a token costs one round of shuffles for two sums.
//
//   general_delta_scan_kernel      steps of single tokens and short portions: inputs made and walked in one kernel
//   general_delta_prepare_kernel   steps with portions: per token and head a row of floats [r | u | w | a | kn, r.(a u), r.k, 0 | v]
//   general_delta_walk_kernel      the walk over the tokens, whose rows arrive by asynchronous copies a chunk ahead
#include "fast_math.cuh"

struct GDeltaArgs {
    const void* r;              // [n, H * dk] rows of T
    const void* k;              // [n, H * dk]
    const void* v;              // [n, H * dv]
    const void* a_pre;          // [n, H * dk]
    const void* z;              // [n, H * dk]
    long long ldr, ldk, ldv, lda, ldz;
    const float* a_bias;        // [H * dk] or null
    const float* z_bias;        // [H * dk] or null
    float* state;               // [slots][H][dk][dv]
    float* out;                 // [n, H * dv] float, row stride ldo
    long long ldo;
    const int* q_start;
    const int* state_slots;
    int H, dk, dv;
    float rate, unit_eps;
    int chunk;                  // tokens staged in shared memory at a time
};

// One or two neighbouring elements of a row.
template <typename T, int VW> __device__ __forceinline__ void gd_load(const T* p, float (&v)[VW]) {
    if constexpr (VW == 2 && sizeof(T) == 2) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
        v[0] = f.x;
        v[1] = f.y;
    } else {
#pragma unroll
        for (int e = 0; e < VW; ++e) v[e] = to_f32<T>(p[e]);
    }
}

// A warp makes one token's inputs of one head: calls put(i, r, u, w, a) for its channels i (VW neighbours at a time, from
// VW * lane on) and returns the three sums to every lane.
template <typename T, int VW, typename Put>
__device__ __forceinline__ void gd_inputs(const GDeltaArgs& A, size_t row, int h, int lane, Put put, float& kn, float& ra, float& rk) {
    const T* rp = (const T*)A.r + row * A.ldr + h * A.dk;
    const T* kp = (const T*)A.k + row * A.ldk + h * A.dk;
    const T* ap = (const T*)A.a_pre + row * A.lda + h * A.dk;
    const T* zp = (const T*)A.z + row * A.ldz + h * A.dk;
    const float* ab = A.a_bias ? A.a_bias + h * A.dk : nullptr;
    const float* zb = A.z_bias ? A.z_bias + h * A.dk : nullptr;
    float ss = 0.0f;
    for (int i = lane * VW; i < A.dk; i += 32 * VW) {
        float x[VW];
        gd_load<T, VW>(kp + i, x);
#pragma unroll
        for (int e = 0; e < VW; ++e) ss = fmaf(x[e], x[e], ss);
    }
    kn = sqrtf(warp_sum(ss) + A.unit_eps);
    const float inv = 1.0f / kn, rate2 = -A.rate * FM_LOG2E;
    float sa = 0.0f, sk = 0.0f;
    for (int i = lane * VW; i < A.dk; i += 32 * VW) {
        float x[VW], r[VW], a[VW], z[VW];
        gd_load<T, VW>(kp + i, x);
        gd_load<T, VW>(rp + i, r);
        gd_load<T, VW>(ap + i, a);
        gd_load<T, VW>(zp + i, z);
#pragma unroll
        for (int e = 0; e < VW; ++e) {
            const float u = x[e] * inv, av = fm_sigmoid(a[e] + (ab ? ab[i + e] : 0.0f));
            const float w = fm_ex2(rate2 * fm_sigmoid(z[e] + (zb ? zb[i + e] : 0.0f)));
            sa = fmaf(r[e], av * u, sa);
            sk = fmaf(r[e], x[e], sk);
            put(i + e, r[e], u, w, av);
        }
    }
    ra = warp_sum(sa);
    rk = warp_sum(sk);
}

// Pairs of channels may be read together: even head sizes and strides, aligned rows.
static bool gd_pairs(const GDeltaArgs& A) {
    return !(A.dk & 1) && !((A.ldr | A.ldk | A.lda | A.ldz) & 1) && !(((uintptr_t)A.r | (uintptr_t)A.k | (uintptr_t)A.a_pre | (uintptr_t)A.z) & 3);
}

// Grid (request, head, tile of DVT value channels).  A thread keeps DKP rows of one column of S in registers; the P threads
// that share a column are neighbouring lanes.  Key channels beyond dk are padded with r = u = a = 0, w = 1.
template <typename T, int DKP>
__global__ void general_delta_scan_kernel(GDeltaArgs A, int P, int DVT) {
    extern __shared__ __align__(16) float sm[];
    const int r = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * DVT;
    const int tid = threadIdx.x, nthreads = blockDim.x, lane = tid & 31, warp = tid >> 5, nwarps = nthreads >> 5;
    const int part = tid % P, cl = tid / P, col = col0 + cl;
    const bool col_ok = cl < DVT && col < A.dv;
    const int TC = A.chunk, pstride = DKP + 4, tstride = P * pstride;
    float* rs = sm;
    float* us = rs + TC * tstride;
    float* ws = us + TC * tstride;
    float* as = ws + TC * tstride;
    float* vs = as + TC * tstride;                // [TC][DVT]
    float* os = vs + TC * DVT;                    // [TC][DVT]
    float* sc = os + TC * DVT;                    // [TC][4]: kn, r.(a u), r.k
    pdl_start();
    const int row0 = A.q_start[r], row1 = A.q_start[r + 1];
    float* st = A.state + (((size_t)A.state_slots[r] * A.H + h) * A.dk) * A.dv;
    float S[DKP];
#pragma unroll
    for (int i = 0; i < DKP; ++i) {
        const int kr = part * DKP + i;
        S[i] = (col_ok && kr < A.dk) ? st[(size_t)kr * A.dv + col] : 0.0f;
    }
    for (int idx = tid; idx < TC * P * DKP; idx += nthreads) {
        const int tt = idx / (P * DKP), i = idx - tt * (P * DKP);
        if (i >= A.dk) {
            const int at = tt * tstride + (i / DKP) * pstride + i % DKP;
            rs[at] = us[at] = as[at] = 0.0f;
            ws[at] = 1.0f;
        }
    }
    for (int c0 = row0; c0 < row1; c0 += TC) {
        const int tc = min(TC, row1 - c0);
        __syncthreads();                          // the chunk before has been read
        for (int tt = warp; tt < tc; tt += nwarps) {
            float kn, ra, rk;
            gd_inputs<T, 1>(A, (size_t)(c0 + tt), h, lane, [&](int i, float rv, float u, float w, float a) {
                const int at = tt * tstride + (i / DKP) * pstride + i % DKP;
                rs[at] = rv;
                us[at] = u;
                ws[at] = w;
                as[at] = a;
            }, kn, ra, rk);
            if (lane == 0) { sc[tt * 4] = kn; sc[tt * 4 + 1] = ra; sc[tt * 4 + 2] = rk; }
        }
        for (int idx = tid; idx < tc * DVT; idx += nthreads) {
            const int tt = idx / DVT, j = idx - tt * DVT, c = col0 + j;
            vs[idx] = c < A.dv ? to_f32<T>(((const T*)A.v)[(size_t)(c0 + tt) * A.ldv + h * A.dv + c]) : 0.0f;
        }
        __syncthreads();
        if (cl < DVT) {
            for (int tt = 0; tt < tc; ++tt) {
                const int at = tt * tstride + part * pstride;
                const float4* r4 = reinterpret_cast<const float4*>(rs + at);
                const float4* u4 = reinterpret_cast<const float4*>(us + at);
                const float4* w4 = reinterpret_cast<const float4*>(ws + at);
                const float4* a4 = reinterpret_cast<const float4*>(as + at);
                float p0 = 0.0f, p1 = 0.0f, q0 = 0.0f, q1 = 0.0f;
#pragma unroll
                for (int i = 0; i < DKP / 4; ++i) {
                    const float4 u = u4[i], w = w4[i], rv = r4[i];
                    p0 = fmaf(S[4 * i], u.x, p0);
                    p1 = fmaf(S[4 * i + 1], u.y, p1);
                    p0 = fmaf(S[4 * i + 2], u.z, p0);
                    p1 = fmaf(S[4 * i + 3], u.w, p1);
                    S[4 * i] *= w.x; S[4 * i + 1] *= w.y; S[4 * i + 2] *= w.z; S[4 * i + 3] *= w.w;
                    q0 = fmaf(S[4 * i], rv.x, q0);
                    q1 = fmaf(S[4 * i + 1], rv.y, q1);
                    q0 = fmaf(S[4 * i + 2], rv.z, q0);
                    q1 = fmaf(S[4 * i + 3], rv.w, q1);
                }
                float p = p0 + p1, q = q0 + q1;
                for (int o = 1; o < P; o <<= 1) {
                    p += __shfl_xor_sync(0xffffffffu, p, o);
                    q += __shfl_xor_sync(0xffffffffu, q, o);
                }
                const float v = vs[tt * DVT + cl], knv = sc[tt * 4] * v;
#pragma unroll
                for (int i = 0; i < DKP / 4; ++i) {
                    const float4 u = u4[i], a = a4[i];
                    S[4 * i] = fmaf(u.x, fmaf(-a.x, p, knv), S[4 * i]);
                    S[4 * i + 1] = fmaf(u.y, fmaf(-a.y, p, knv), S[4 * i + 1]);
                    S[4 * i + 2] = fmaf(u.z, fmaf(-a.z, p, knv), S[4 * i + 2]);
                    S[4 * i + 3] = fmaf(u.w, fmaf(-a.w, p, knv), S[4 * i + 3]);
                }
                if (part == 0) os[tt * DVT + cl] = fmaf(sc[tt * 4 + 2], v, fmaf(-sc[tt * 4 + 1], p, q));
            }
        }
        __syncthreads();
        for (int idx = tid; idx < tc * DVT; idx += nthreads) {
            const int tt = idx / DVT, j = idx - tt * DVT, c = col0 + j;
            if (c < A.dv) A.out[(size_t)(c0 + tt) * A.ldo + h * A.dv + c] = os[idx];
        }
    }
#pragma unroll
    for (int i = 0; i < DKP; ++i) {
        const int kr = part * DKP + i;
        if (col_ok && kr < A.dk) st[(size_t)kr * A.dv + col] = S[i];
    }
}

// A (token, head) row of the prepared inputs: r, u, w and a of dk channels each, padded to a multiple of 4 by channels that do
// nothing, then kn, r.(a u), r.k, 0, then v, padded.  Its size in floats (ops.py has the same formula).
__host__ __device__ static inline int gd_pad4(int n) { return (n + 3) / 4 * 4; }
__host__ __device__ static inline int gd_work_row(int dk, int dv) { return 4 * gd_pad4(dk) + 4 + gd_pad4(dv); }

template <typename T, int VW>
__global__ void __launch_bounds__(128) general_delta_prepare_kernel(GDeltaArgs A, float* __restrict__ work) {
    // The walk's CTAs come when all of these have ended: placed while these fill the SMs, they would crowd on a few.
    pdl_wait();
    const int lane = threadIdx.x & 31, row = blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), dk = A.dk, d4 = gd_pad4(dk);
    if (h >= A.H) return;
    float* w = work + ((size_t)row * A.H + h) * gd_work_row(dk, A.dv);
    float kn, ra, rk;
    gd_inputs<T, VW>(A, (size_t)row, h, lane, [&](int i, float rv, float u, float wv, float a) {
        w[i] = rv;
        w[d4 + i] = u;
        w[2 * d4 + i] = wv;
        w[3 * d4 + i] = a;
    }, kn, ra, rk);
    if (lane < d4 - dk) {
        w[dk + lane] = w[d4 + dk + lane] = w[3 * d4 + dk + lane] = 0.0f;
        w[2 * d4 + dk + lane] = 1.0f;
    }
    if (lane < 4) w[4 * d4 + lane] = lane == 0 ? kn : lane == 1 ? ra : lane == 2 ? rk : 0.0f;
    const T* vp = (const T*)A.v + (size_t)row * A.ldv + h * A.dv;
    for (int i = lane; i < gd_pad4(A.dv); i += 32) w[4 * d4 + 4 + i] = i < A.dv ? to_f32<T>(vp[i]) : 0.0f;
}

__device__ __forceinline__ void gd_copy16(uint32_t dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}

// Grid (request, head, tile of DVT value channels).  P lanes of a warp share GD_COLS neighbouring columns of S, of which a
// thread keeps DKP rows each, two rows to a register pair: a token's row values are read from shared memory once for both
// columns.  (The walk is bound by the chain sum -> update of one token after another; one column a thread with twice the warps
// measured a tenth slower.)  The sums u . S that the update waits for go round the lanes at once; the read-outs of four tokens
// wait and are summed together, each round of shuffles handing half of them over.  Chunks of TC tokens' rows arrive by asynchronous copies a chunk ahead; tokens
// beyond the portion's end are rows that leave S as it is.
constexpr int GD_COLS = 2, GD_GROUP = 4, GD_WARPS = 4 / GD_COLS;

template <int DKP, int P>
__global__ void __launch_bounds__(32 * GD_WARPS) general_delta_walk_kernel(GDeltaArgs A, const float* __restrict__ work) {
    constexpr int CW = 32 / P * GD_COLS, DVT = CW * GD_WARPS, THREADS = 32 * GD_WARPS, PS = DKP + 4, TS = P * PS, V = GD_COLS * GD_GROUP;
    extern __shared__ __align__(16) float sm[];
    pdl_start();
    const int r = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * DVT;
    const int tid = threadIdx.x, lane = tid & 31, part = lane % P, cl = (tid >> 5) * CW + lane / P * GD_COLS, col = col0 + cl;
    const int dk = A.dk, TC = A.chunk, wrow = gd_work_row(dk, A.dv);
    // two buffers of a chunk's rows: [r, u, w, a: TC x TS each][v: TC x DVT][kn, r.(a u), r.k: TC x 4], then the outputs [TC x DVT]
    const int buf_floats = TC * (4 * TS + DVT + 4);
    float* os = sm + 2 * buf_floats;
    const int row0 = A.q_start[r], row1 = A.q_start[r + 1];
    if (row0 >= row1) return;
    float* st = A.state + (((size_t)A.state_slots[r] * A.H + h) * dk) * A.dv;
    f32x2 S[GD_COLS][DKP / 2];
#pragma unroll
    for (int c = 0; c < GD_COLS; ++c)
#pragma unroll
        for (int i = 0; i < DKP / 2; ++i) {
            const int kr = part * DKP + 2 * i;
            const bool ok = col + c < A.dv;
            S[c][i] = pack2f(ok && kr < dk ? st[(size_t)kr * A.dv + col + c] : 0.0f, ok && kr + 1 < dk ? st[(size_t)(kr + 1) * A.dv + col + c] : 0.0f);
        }
    // Channels beyond the padded head (r = u = a = 0, w = 1) are written once; whole tokens beyond the end in the last chunk.
    const int d4 = gd_pad4(dk);
    auto neutral = [&](float* base, int tt, int i) {
        float* at = base + tt * TS + (i / DKP) * PS + i % DKP;
        at[0] = 0.0f;
        at[TC * TS] = 0.0f;
        at[2 * TC * TS] = 1.0f;
        at[3 * TC * TS] = 0.0f;
    };
    if (d4 < P * DKP) {
        for (int idx = tid; idx < 2 * TC * P * DKP; idx += THREADS) {
            const int b = idx / (TC * P * DKP), rest = idx - b * (TC * P * DKP);
            const int tt = rest / (P * DKP), i = rest - tt * (P * DKP);
            if (i >= d4) neutral(sm + b * buf_floats, tt, i);
        }
    }
    // A token's pieces of 16 bytes: four vectors of P * DKP / 4, the scalars, DVT / 4 of v.  Every thread has fixed pieces of
    // every token and walks their addresses from token to token.
    constexpr int VEC_PIECES = P * DKP, PIECES = VEC_PIECES + 1 + DVT / 4, MINE = (PIECES + THREADS - 1) / THREADS;
    const float* src[MINE];
    int dst[MINE], step[MINE];
#pragma unroll
    for (int k = 0; k < MINE; ++k) {
        const int piece = tid + k * THREADS;
        src[k] = nullptr;
        dst[k] = step[k] = 0;
        const float* w = work + ((size_t)row0 * A.H + h) * wrow;
        if (piece < VEC_PIECES) {
            const int which = piece / (P * DKP / 4), i = (piece - which * (P * DKP / 4)) * 4;
            if (i < d4) {
                src[k] = w + which * d4 + i;
                dst[k] = which * TC * TS + (i / DKP) * PS + i % DKP;
                step[k] = TS;
            }
        } else if (piece == VEC_PIECES) {
            src[k] = w + 4 * d4;
            dst[k] = TC * (4 * TS + DVT);
            step[k] = 4;
        } else if (piece < PIECES) {
            const int j = (piece - VEC_PIECES - 1) * 4;
            if (col0 + j < A.dv) {
                src[k] = w + 4 * d4 + 4 + col0 + j;
                dst[k] = 4 * TC * TS + j;
                step[k] = DVT;
            }
        }
    }
    const uint32_t sm0 = (uint32_t)__cvta_generic_to_shared(sm);
    const size_t token = (size_t)A.H * wrow;
    auto fetch = [&](int c0, int b) {
        const int tc = min(TC, row1 - c0);
        float* base = sm + b * buf_floats;
#pragma unroll
        for (int k = 0; k < MINE; ++k) {
            if (!src[k]) continue;
            uint32_t to = sm0 + 4u * (uint32_t)(b * buf_floats + dst[k]);
            const float* from = src[k];
            for (int tt = 0; tt < tc; ++tt) {
                gd_copy16(to, from);
                to += 4u * (uint32_t)step[k];
                from += token;
            }
            src[k] = from;
        }
        if (tc < TC) {
            float* vs = base + 4 * TC * TS;
            float* sc = vs + TC * DVT;
            for (int idx = tid; idx < (TC - tc) * P * DKP; idx += THREADS) neutral(base, tc + idx / (P * DKP), idx % (P * DKP));
            for (int idx = tc * DVT + tid; idx < TC * DVT; idx += THREADS) vs[idx] = 0.0f;
            for (int idx = tc * 4 + tid; idx < TC * 4; idx += THREADS) sc[idx] = 0.0f;
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(row0, 0);
    int b = 0;
    for (int c0 = row0; c0 < row1; c0 += TC, b ^= 1) {
        const int tc = min(TC, row1 - c0);
        if (c0 + TC < row1) {
            fetch(c0 + TC, b ^ 1);                 // its buffer was walked two chunks ago; the barriers since cover it
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();                           // everybody's copies of this chunk have landed; the outputs before are stored
        const float* mine = sm + b * buf_floats + part * PS;
        const float* vs = sm + b * buf_floats + 4 * TC * TS;
        const float* sc = vs + TC * DVT;
        for (int g = 0; g < tc; g += GD_GROUP) {
            float q[V];
#pragma unroll
            for (int k = 0; k < GD_GROUP; ++k) {
                const int tt = g + k;
                const float4 s4 = *reinterpret_cast<const float4*>(sc + tt * 4);
                float v[GD_COLS];
#pragma unroll
                for (int c = 0; c < GD_COLS; ++c) v[c] = col + c < A.dv ? vs[tt * DVT + cl + c] : 0.0f;
                f32x2 u[DKP / 2], w[DKP / 2], rv[DKP / 2], av[DKP / 2];
                auto read = [&](f32x2 (&x)[DKP / 2], int which) {
#pragma unroll
                    for (int i = 0; i < DKP / 4; ++i) {
                        const float4 f = reinterpret_cast<const float4*>(mine + which * TC * TS + tt * TS)[i];
                        x[2 * i] = pack2f(f.x, f.y);
                        x[2 * i + 1] = pack2f(f.z, f.w);
                    }
                };
                read(u, 1);
                read(w, 2);
                read(rv, 0);
                read(av, 3);
                float p[GD_COLS];
#pragma unroll
                for (int c = 0; c < GD_COLS; ++c) {
                    f32x2 x = mul2f(S[c][0], u[0]), y = mul2f(S[c][1], u[1]);
#pragma unroll
                    for (int i = 2; i < DKP / 2; i += 2) { x = fma2f(S[c][i], u[i], x); y = fma2f(S[c][i + 1], u[i + 1], y); }
                    p[c] = sum2f(x) + sum2f(y);
                }
#pragma unroll
                for (int o = 1; o < P; o <<= 1)
#pragma unroll
                    for (int c = 0; c < GD_COLS; ++c) p[c] += __shfl_xor_sync(0xffffffffu, p[c], o);
#pragma unroll
                for (int c = 0; c < GD_COLS; ++c) {
                    f32x2 x = pack2f(0.0f, 0.0f), y = x;
#pragma unroll
                    for (int i = 0; i < DKP / 2; i += 2) {
                        S[c][i] = mul2f(S[c][i], w[i]);
                        S[c][i + 1] = mul2f(S[c][i + 1], w[i + 1]);
                        x = fma2f(S[c][i], rv[i], x);
                        y = fma2f(S[c][i + 1], rv[i + 1], y);
                    }
                    // the token's own terms join the sum in one of the lanes
                    q[k * GD_COLS + c] = sum2f(x) + sum2f(y) + (part == 0 ? fmaf(s4.z, v[c], -s4.y * p[c]) : 0.0f);
                    const f32x2 mp = pack2f(-p[c], -p[c]), kv = pack2f(s4.x * v[c], s4.x * v[c]);
#pragma unroll
                    for (int i = 0; i < DKP / 2; ++i) S[c][i] = fma2f(u[i], fma2f(av[i], mp, kv), S[c][i]);
                }
            }
            // V sums over P lanes: halve the values while there are several, then add up what is left
            int first = 0;                          // which of the V values this lane's first one is
            constexpr int ROUNDS_DEALT = P >= V ? V : P;
            int left = V;
#pragma unroll
            for (int o = 1; o < ROUNDS_DEALT; o <<= 1) {
                const bool upper = part & o;
                left >>= 1;
#pragma unroll
                for (int i = 0; i < V / 2; ++i)
                    if (i < left) {
                        const float keep = upper ? q[i + left] : q[i], give = upper ? q[i] : q[i + left];
                        q[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                    }
                if (upper) first += left;
            }
#pragma unroll
            for (int o = ROUNDS_DEALT; o < P; o <<= 1) q[0] += __shfl_xor_sync(0xffffffffu, q[0], o);
            constexpr int EACH = V / ROUNDS_DEALT;
            if (part < ROUNDS_DEALT) {
#pragma unroll
                for (int i = 0; i < EACH; ++i) {
                    const int which = first + i;
                    os[(g + which / GD_COLS) * DVT + cl + which % GD_COLS] = q[i];
                }
            }
        }
        __syncthreads();
        for (int idx = tid; idx < tc * DVT; idx += THREADS) {
            const int tt = idx / DVT, j = idx - tt * DVT, c = col0 + j;
            if (c < A.dv) A.out[(size_t)(c0 + tt) * A.ldo + h * A.dv + c] = os[idx];
        }
    }
#pragma unroll
    for (int c = 0; c < GD_COLS; ++c)
#pragma unroll
        for (int i = 0; i < DKP / 2; ++i) {
            const int kr = part * DKP + 2 * i;
            float x, y;
            unpack2f(S[c][i], x, y);
            if (col + c < A.dv && kr < dk) st[(size_t)kr * A.dv + col + c] = x;
            if (col + c < A.dv && kr + 1 < dk) st[(size_t)(kr + 1) * A.dv + col + c] = y;
        }
}

constexpr int GD_WALK_SMEM = 100 * 1024;

template <int DKP, int P>
static int launch_gd_walk(GDeltaArgs A, int n_reqs, const float* work, cudaStream_t s) {
    constexpr int DVT = 32 / P * GD_COLS * GD_WARPS;
    auto bytes = [&](int tc) { return (size_t)tc * (2 * (4 * P * (DKP + 4) + DVT + 4) + DVT) * sizeof(float); };
    int chunk = 16;
    while (chunk > GD_GROUP && bytes(chunk) > GD_WALK_SMEM) chunk >>= 1;
    if (bytes(chunk) > GD_WALK_SMEM) return VCB_ERR_UNSUPPORTED;
    static unsigned long long configured = 0;
    if (int e = vcb_allow_dynamic_smem(general_delta_walk_kernel<DKP, P>, GD_WALK_SMEM, &configured)) return e;
    A.chunk = chunk;
    dim3 grid(n_reqs, A.H, (A.dv + DVT - 1) / DVT);
    vcb_launch(general_delta_walk_kernel<DKP, P>, grid, 32 * GD_WARPS, bytes(chunk), s, A, work);
    return vcb_last_error();
}

template <typename T>
static int launch_gd_scan(const GDeltaArgs& A, int n_reqs, cudaStream_t s) {
    const int dkp = A.dk <= 32 ? 8 : A.dk <= 64 ? 16 : 32;
    int P = 1;
    while (P * dkp < A.dk) P <<= 1;
    if (P > 32) return VCB_ERR_UNSUPPORTED;
    const int dvt = P <= 8 ? 32 : 256 / P;
    const int threads = ((dvt * P + 31) / 32) * 32;
    int chunk = 8;
    auto bytes = [&](int tc) { return ((size_t)tc * (4 * P * (dkp + 4) + 2 * dvt + 4)) * sizeof(float); };
    while (chunk > 1 && bytes(chunk) > 48 * 1024) chunk >>= 1;
    GDeltaArgs B = A;
    B.chunk = chunk;
    dim3 grid(n_reqs, A.H, (A.dv + dvt - 1) / dvt);
    if (dkp == 8) vcb_launch(general_delta_scan_kernel<T, 8>, grid, threads, bytes(chunk), s, B, P, dvt);
    else if (dkp == 16) vcb_launch(general_delta_scan_kernel<T, 16>, grid, threads, bytes(chunk), s, B, P, dvt);
    else vcb_launch(general_delta_scan_kernel<T, 32>, grid, threads, bytes(chunk), s, B, P, dvt);
    return vcb_last_error();
}

template <typename T>
static int launch_gd_portions(const GDeltaArgs& A, int n_reqs, int n_tokens, float* work, cudaStream_t s) {
    if (A.dk > 512) return launch_gd_scan<T>(A, n_reqs, s);     // very long keys: the kernel above
    if (gd_pairs(A)) vcb_launch(general_delta_prepare_kernel<T, 2>, dim3(n_tokens, (A.H + 3) / 4), 128, 0, s, A, work);
    else vcb_launch(general_delta_prepare_kernel<T, 1>, dim3(n_tokens, (A.H + 3) / 4), 128, 0, s, A, work);
    if (int e = vcb_last_error()) return e;
    if (A.dk <= 8) return launch_gd_walk<8, 1>(A, n_reqs, work, s);
    if (A.dk <= 16) return launch_gd_walk<8, 2>(A, n_reqs, work, s);
    if (A.dk <= 32) return launch_gd_walk<8, 4>(A, n_reqs, work, s);
    if (A.dk <= 64) return launch_gd_walk<8, 8>(A, n_reqs, work, s);
    if (A.dk <= 128) return launch_gd_walk<8, 16>(A, n_reqs, work, s);
    if (A.dk <= 256) return launch_gd_walk<8, 32>(A, n_reqs, work, s);
    return launch_gd_walk<16, 32>(A, n_reqs, work, s);
}

VCB_EXPORT int vcb_general_delta(const void* r, long long ldr, const void* k, long long ldk, const void* v, long long ldv,
                                 const void* a_pre, long long lda, const void* z, long long ldz, const float* a_bias, const float* z_bias,
                                 float* state, float* out, long long ldo, const int* q_start, const int* state_slots, int n_reqs, int H,
                                 int dk, int dv, float rate, float unit_eps, float* work, int n_tokens, int dtype, void* stream) {
    if (n_reqs <= 0) return 0;
    if (!r || !k || !v || !a_pre || !z || !state || !out || H <= 0 || dk <= 0 || dv <= 0 || H > 65535 || (dv + 7) / 8 > 65535) return VCB_ERR_BAD_ARG;
    GDeltaArgs A{r, k, v, a_pre, z, ldr, ldk, ldv, lda, ldz, a_bias, z_bias, state, out, ldo, q_start, state_slots, H, dk, dv, rate, unit_eps, 0};
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype != VCB_F32 && dtype != VCB_BF16) return VCB_ERR_BAD_ARG;
    if (work && n_tokens > 0)
        return dtype == VCB_F32 ? launch_gd_portions<float>(A, n_reqs, n_tokens, work, s) : launch_gd_portions<__nv_bfloat16>(A, n_reqs, n_tokens, work, s);
    return dtype == VCB_F32 ? launch_gd_scan<float>(A, n_reqs, s) : launch_gd_scan<__nv_bfloat16>(A, n_reqs, s);
}

// ------------------------------------------------------------------------------- out = tanh(x), rows of T
template <typename T>
__global__ void tanh_rows_kernel(const T* __restrict__ x, long long ldx, T* __restrict__ out, long long ldo, int n, int width) {
    pdl_start();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < (long long)n * width; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / width;
        const int c = (int)(i - t * width);
        out[t * ldo + c] = from_f32<T>(tanhf(to_f32<T>(x[t * ldx + c])));
    }
}

VCB_EXPORT int vcb_tanh_rows(const void* x, long long ldx, void* out, long long ldo, int n, int width, int dtype, void* stream) {
    if (n <= 0 || width <= 0) return 0;
    if (!x || !out) return VCB_ERR_BAD_ARG;
    const long long total = (long long)n * width;
    const int blocks = (int)((total + 255) / 256 < vcb_sm_count() * 8 ? (total + 255) / 256 : vcb_sm_count() * 8);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == VCB_F32) vcb_launch(tanh_rows_kernel<float>, blocks, 256, 0, s, (const float*)x, ldx, (float*)out, ldo, n, width);
    else if (dtype == VCB_BF16) vcb_launch(tanh_rows_kernel<__nv_bfloat16>, blocks, 256, 0, s, (const __nv_bfloat16*)x, ldx, (__nv_bfloat16*)out, ldo, n, width);
    else return VCB_ERR_BAD_ARG;
    return vcb_last_error();
}
