// A matrix per head that decays by one number per token and takes up an outer product, its inputs shared by groups of heads:
//
//     S_t = e_t S_(t-1) + B_t (dt_t x_t)^T      e_t = 2^(a2_h dt_t),  dt_t = softplus(dt_pre_t + dt_bias_h)      S: [N, P] float
//     y_t = S_t^T C_t + d_h x_t                                                                                  y: float
//
// x [n, H * P], B and C [n, G * N] are rows of the activations' type (head h reads group h / (H / G)), dt_pre [n, H] too; step
// sizes, decays, state and sums are float.  The state lives in the request's slot ([slots][H][N][P]), is read at the start of a
// request's portion and left there at its end.
//
//   state_dual_walk_kernel    walks a request's tokens one by one with S in registers: single tokens, short portions, float32
//   state_dual_chunk_kernel   bfloat16 portions on tensor cores, 64 tokens at a time.  With A_t the sum of a2 dt over the chunk's
//                             tokens up to t, the same recurrence is
//                               y_t = 2^(A_t) S^T C_t + sum_(s <= t) 2^(A_t - A_s) dt_s (C_t . B_s) x_s
//                               S  <- 2^(A_last) S + sum_s B_s (2^(A_last - A_s) dt_s x_s)^T
//                             that is four products.  B, C and x enter them as they are; what is float (the state, the weighted
//                             scores, the weighted x) enters as three bfloat16 terms, which hold all 24 bits.  Exponents are
//                             differences of sums, at most zero: nothing is divided by a decay.
//
// The reference has no recurrent mixer.
#include "fast_math.cuh"

struct DualArgs {
    const void* x;              // [n, H * P] rows of T
    const void* b;              // [n, G * N]
    const void* c;              // [n, G * N]
    const void* dt_pre;         // [n, H]
    long long ldx, ldb, ldc, lddt;
    const float* dt_bias;       // [H]
    const float* a2;            // [H]: the decay's rate times log2(e), negative
    const float* d;             // [H]
    float* state;               // [slots][H][N][P]
    float* y;                   // [n, H * P]
    long long ldy;
    const int* q_start;
    const int* state_slots;
    int H, G, N, P;
};

__device__ __forceinline__ float sd_softplus(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

// ------------------------------------------------------------------------------------------- walk
// Grid (tiles of columns, heads, requests); block (CX, RG): thread (x, y) keeps rows y, y + RG, ... of the columns VW x .. of its
// tile.  TC tokens are staged together; their partial read-outs are summed over the row groups at the end of the chunk.
#define SDW_TC 8

template <typename T, int VW, int R>
__global__ void __launch_bounds__(512) state_dual_walk_kernel(DualArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int CX = blockDim.x, RG = blockDim.y, CT = CX * VW, tid = threadIdx.y * CX + threadIdx.x, nthreads = CX * RG;
    const int h = blockIdx.y, r = blockIdx.z, col0 = blockIdx.x * CT;
    const int NP = RG * R;
    float* xs = sm;                          // [TC][CT]
    float* bs = xs + SDW_TC * CT;            // [TC][NP]
    float* cs = bs + SDW_TC * NP;
    float* ts = cs + SDW_TC * NP;            // [TC][2]: decay, step
    float* ps = ts + SDW_TC * 2;             // [TC][RG][CT]
    const int row0 = a.q_start[r], row1 = a.q_start[r + 1];        // the step's index arrays are older than the kernel before
    const int col = col0 + threadIdx.x * VW;
    const bool there = col < a.P;            // P is a multiple of VW
    const float a2 = a.a2[h], bias = a.dt_bias[h], dh = a.d[h];
    float* st = a.state + ((size_t)a.state_slots[r] * a.H + h) * a.N * a.P;
    const int g = h / (a.H / a.G);
    pdl_start();
    float S[R][VW];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int n = threadIdx.y + i * RG;
        if (VW == 4 && there && n < a.N) {
            const float4 q = *reinterpret_cast<const float4*>(st + (size_t)n * a.P + col);
            S[i][0] = q.x;
            if (VW == 4) { S[i][VW > 1 ? 1 : 0] = q.y; S[i][VW > 2 ? 2 : 0] = q.z; S[i][VW > 3 ? 3 : 0] = q.w; }
        } else {
#pragma unroll
            for (int e = 0; e < VW; ++e) S[i][e] = there && n < a.N ? st[(size_t)n * a.P + col + e] : 0.0f;
        }
    }
    const T* xp = (const T*)a.x + (size_t)h * a.P;
    const T* bp = (const T*)a.b + (size_t)g * a.N;
    const T* cp = (const T*)a.c + (size_t)g * a.N;
    for (int t0 = row0; t0 < row1; t0 += SDW_TC) {
        const int tc = min(SDW_TC, row1 - t0);
        if (t0 > row0) __syncthreads();      // the chunk before has been read
        for (int i = tid; i < tc * CT; i += nthreads) {
            const int t = i / CT, c = col0 + i - t * CT;
            xs[i] = c < a.P ? to_f32<T>(xp[(size_t)(t0 + t) * a.ldx + c]) : 0.0f;
        }
        for (int i = tid; i < tc * NP; i += nthreads) {
            const int t = i / NP, n = i - t * NP;
            bs[i] = n < a.N ? to_f32<T>(bp[(size_t)(t0 + t) * a.ldb + n]) : 0.0f;
            cs[i] = n < a.N ? to_f32<T>(cp[(size_t)(t0 + t) * a.ldc + n]) : 0.0f;
        }
        for (int t = tid; t < tc; t += nthreads) {
            const float dt = sd_softplus(to_f32<T>(((const T*)a.dt_pre)[(size_t)(t0 + t) * a.lddt + h]) + bias);
            ts[2 * t] = exp2f(a2 * dt);
            ts[2 * t + 1] = dt;
        }
        __syncthreads();
        for (int t = 0; t < tc; ++t) {
            const float decay = ts[2 * t], dt = ts[2 * t + 1];
            float dx[VW], y[VW];
#pragma unroll
            for (int e = 0; e < VW; ++e) { dx[e] = dt * xs[t * CT + threadIdx.x * VW + e]; y[e] = 0.0f; }
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const float bn = bs[t * NP + threadIdx.y + i * RG], cn = cs[t * NP + threadIdx.y + i * RG];
#pragma unroll
                for (int e = 0; e < VW; ++e) {
                    S[i][e] = fmaf(decay, S[i][e], bn * dx[e]);
                    y[e] = fmaf(S[i][e], cn, y[e]);
                }
            }
#pragma unroll
            for (int e = 0; e < VW; ++e) ps[(t * RG + threadIdx.y) * CT + threadIdx.x * VW + e] = y[e];
        }
        __syncthreads();
        for (int i = tid; i < tc * CT; i += nthreads) {
            const int t = i / CT, j = i - t * CT;
            if (col0 + j >= a.P) continue;
            float s = 0.0f;
            for (int k = 0; k < RG; ++k) s += ps[(t * RG + k) * CT + j];
            a.y[(size_t)(t0 + t) * a.ldy + (size_t)h * a.P + col0 + j] = fmaf(dh, xs[i], s);
        }
    }
    if (!there) return;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int n = threadIdx.y + i * RG;
        if (n >= a.N) continue;
        if (VW == 4) *reinterpret_cast<float4*>(st + (size_t)n * a.P + col) = make_float4(S[i][0], S[i][VW > 1 ? 1 : 0], S[i][VW > 2 ? 2 : 0], S[i][VW > 3 ? 3 : 0]);
        else st[(size_t)n * a.P + col] = S[i][0];
    }
}

template <typename T, int VW, int R>
static int launch_walk_as(const DualArgs& a, int n_reqs, cudaStream_t s) {
    const int RG = (a.N + R - 1) / R;
    int CX = VW == 4 ? 16 : 32;
    while (CX > 4 && (CX / 2) * VW >= a.P) CX /= 2;
    while (CX * RG > 512) CX /= 2;
    const int CT = CX * VW;
    const size_t smem = (size_t)SDW_TC * (CT + 2 * RG * R + 2 + RG * CT) * sizeof(float);
    static unsigned long long configured = 0;
    if (smem > 48 * 1024) {
        if (smem > 200 * 1024) return VCB_ERR_UNSUPPORTED;
        if (int e = vcb_allow_dynamic_smem(state_dual_walk_kernel<T, VW, R>, 200 * 1024, &configured)) return e;
    }
    vcb_launch(state_dual_walk_kernel<T, VW, R>, dim3((a.P + CT - 1) / CT, a.H, n_reqs), dim3(CX, RG), smem, s, a);
    return vcb_last_error();
}

template <typename T>
static int launch_walk(const DualArgs& a, int n_reqs, cudaStream_t s) {
    const bool quads = a.P % 4 == 0;
    if (a.N <= 128) return quads ? launch_walk_as<T, 4, 8>(a, n_reqs, s) : launch_walk_as<T, 1, 8>(a, n_reqs, s);
    if (a.N <= 256) return quads ? launch_walk_as<T, 4, 16>(a, n_reqs, s) : launch_walk_as<T, 1, 16>(a, n_reqs, s);
    return quads ? launch_walk_as<T, 4, 32>(a, n_reqs, s) : launch_walk_as<T, 1, 32>(a, n_reqs, s);
}

// ------------------------------------------------------------------------------------------ chunks
#define SDC_Q 64                 // tokens of a chunk
#define SDC_THREADS 256

__device__ __forceinline__ uint32_t sd_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void sd_copy16(uint32_t dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void sd_ldm(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sd_ldm_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sd_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// A pair of floats as three pairs of bfloat16 whose sum is the pair (each term takes eight bits more of the mantissa).
__device__ __forceinline__ void sd_split3(float u, float v, uint32_t (&t)[3]) {
#pragma unroll
    for (int k = 0; k < 3; ++k) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(u, v);
        t[k] = *reinterpret_cast<const uint32_t*>(&h);
        u -= __low2float(h);
        v -= __high2float(h);
    }
}

// NP: N padded; PT: columns of S a CTA takes.  Rows in shared memory are padded by 16 bytes against bank conflicts.
template <int NP, int PT> struct DualShape {
    static constexpr int LDN = NP + 8, LDP = PT + 8;
    static constexpr int STAGE = SDC_Q * (2 * LDN + LDP);                    // C, B, x of a chunk (elements)
    static constexpr int TERMS = 3 * (NP + SDC_Q) * LDP;                     // the state's and the weighted x's terms
    static constexpr int FLOATS = 2 * 3 * SDC_Q;                             // A, dt, weights; two chunks
    static constexpr int BYTES = (2 * STAGE + TERMS) * 2 + FLOATS * 4;
    static constexpr int ROW_TILES = NP / 16, COL_PARTS = 8 / ROW_TILES;     // how eight warps share S
    static constexpr int SCOLS = PT / COL_PARTS, SB = SCOLS / 8;
    static constexpr int YB = PT / 16;                                       // 8-column blocks of a warp's half of y
};

template <int NP, int PT>
__global__ void __launch_bounds__(SDC_THREADS) state_dual_chunk_kernel(DualArgs a) {
    using Sh = DualShape<NP, PT>;
    constexpr int LDN = Sh::LDN, LDP = Sh::LDP, SB = Sh::SB, YB = Sh::YB;
    extern __shared__ __align__(16) unsigned char smem[];
    __nv_bfloat16* stages = reinterpret_cast<__nv_bfloat16*>(smem);
    __nv_bfloat16* sterm = stages + 2 * Sh::STAGE;                           // [3][NP][LDP]
    __nv_bfloat16* xterm = sterm + 3 * NP * LDP;                             // [3][Q][LDP]
    float* fl = reinterpret_cast<float*>(xterm + 3 * SDC_Q * LDP);           // [2][3][Q]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y, r = blockIdx.z, p0 = blockIdx.x * PT, g = h / (a.H / a.G);
    const int row0 = a.q_start[r], len = a.q_start[r + 1] - row0;
    const float a2 = a.a2[h], bias = a.dt_bias[h], dh = a.d[h];
    float* st = a.state + ((size_t)a.state_slots[r] * a.H + h) * a.N * a.P;
    pdl_start();
    if (len <= 0) return;
    const __nv_bfloat16* xp = (const __nv_bfloat16*)a.x + (size_t)row0 * a.ldx + (size_t)h * a.P + p0;
    const __nv_bfloat16* bp = (const __nv_bfloat16*)a.b + (size_t)row0 * a.ldb + (size_t)g * a.N;
    const __nv_bfloat16* cp = (const __nv_bfloat16*)a.c + (size_t)row0 * a.ldc + (size_t)g * a.N;
    const __nv_bfloat16* dp = (const __nv_bfloat16*)a.dt_pre + (size_t)row0 * a.lddt + h;

    auto load_stage = [&](int t0, int buf) {          // C | B | x of tokens t0 .. of the portion; what is not there arrives as zeros
        const uint32_t cs = sd_smem(stages + buf * Sh::STAGE), bs = cs + SDC_Q * LDN * 2, xs = bs + SDC_Q * LDN * 2;
        constexpr int CN = NP / 8, CPX = PT / 8;
        for (int i = tid; i < SDC_Q * CN; i += SDC_THREADS) {
            const int t = i / CN, n = (i % CN) * 8;
            const bool ok = t0 + t < len && n < a.N;
            sd_copy16(cs + (t * LDN + n) * 2, ok ? cp + (size_t)(t0 + t) * a.ldc + n : cp, ok);
            sd_copy16(bs + (t * LDN + n) * 2, ok ? bp + (size_t)(t0 + t) * a.ldb + n : bp, ok);
        }
        for (int i = tid; i < SDC_Q * CPX; i += SDC_THREADS) {
            const int t = i / CPX, p = (i % CPX) * 8;
            const bool ok = t0 + t < len && p0 + p < a.P;
            sd_copy16(xs + (t * LDP + p) * 2, ok ? xp + (size_t)(t0 + t) * a.ldx + p : bp, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_stage(0, 0);
    float pre[2];                                     // warp 0: dt_pre of tokens lane and lane + 32 of the chunk that comes
    auto fetch_dt = [&](int t0) {
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int t = t0 + lane + 32 * k;
            pre[k] = t < len ? __bfloat162float(dp[(size_t)t * a.lddt]) : 0.0f;
        }
    };
    if (warp == 0) fetch_dt(0);

    // this warp's part of S: rows 16 * rt .. + 15, columns SCOLS * part ..; fragment (row lane / 4 [+ 8], columns (lane % 4) * 2, + 1)
    const int rt = warp % Sh::ROW_TILES, sc0 = (warp / Sh::ROW_TILES) * Sh::SCOLS;
    const int sr = rt * 16 + (lane >> 2), sq = sc0 + (lane & 3) * 2;
    float S[SB][4];
    auto keep_terms = [&]() {                         // S into shared memory as three terms
#pragma unroll
        for (int j = 0; j < SB; ++j) {
            uint32_t lo[3], hi[3];
            sd_split3(S[j][0], S[j][1], lo);
            sd_split3(S[j][2], S[j][3], hi);
#pragma unroll
            for (int k = 0; k < 3; ++k) {
                *reinterpret_cast<uint32_t*>(sterm + (k * NP + sr) * LDP + sq + 8 * j) = lo[k];
                *reinterpret_cast<uint32_t*>(sterm + (k * NP + sr + 8) * LDP + sq + 8 * j) = hi[k];
            }
        }
    };
#pragma unroll
    for (int j = 0; j < SB; ++j) {
        const int c = p0 + sq + 8 * j;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int n = sr + 8 * half;
            const float2 v = n < a.N && c < a.P ? *reinterpret_cast<const float2*>(st + (size_t)n * a.P + c) : make_float2(0.0f, 0.0f);
            S[j][2 * half] = v.x;
            S[j][2 * half + 1] = v.y;
        }
    }
    keep_terms();

    const int tr = (warp & 3) * 16, yc = (warp >> 2) * (PT / 2);       // this warp's 16 tokens and half of the columns of y
    const int lrow = lane & 7, lmat = lane >> 3;                       // row and matrix of an ldmatrix lane
    for (int t0 = 0, it = 0; t0 < len; t0 += SDC_Q, ++it) {
        const int buf = it & 1;
        float* A = fl + buf * 3 * SDC_Q;                               // sums of a2 dt
        float* dt = A + SDC_Q;
        float* we = dt + SDC_Q;                                        // 2^(A_last - A_t) dt_t
        if (warp == 0) {
            float d[2], s[2];
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                d[k] = t0 + lane + 32 * k < len ? sd_softplus(pre[k] + bias) : 0.0f;      // a token that is not there changes nothing
                s[k] = a2 * d[k];
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const float up = __shfl_up_sync(0xffffffffu, s[k], o);
                    if (lane >= o) s[k] += up;
                }
            }
            s[1] += __shfl_sync(0xffffffffu, s[0], 31);
            const float last = __shfl_sync(0xffffffffu, s[1], 31);
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                A[lane + 32 * k] = s[k];
                dt[lane + 32 * k] = d[k];
                we[lane + 32 * k] = fm_ex2(last - s[k]) * d[k];
            }
            if (t0 + SDC_Q < len) fetch_dt(t0 + SDC_Q);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                               // the chunk has landed, its numbers and the state's terms are there
        if (t0 + SDC_Q < len) load_stage(t0 + SDC_Q, buf ^ 1);         // the buffer whose chunk everyone has left
        const __nv_bfloat16* csm = stages + buf * Sh::STAGE;
        const __nv_bfloat16* bsm = csm + SDC_Q * LDN;
        const __nv_bfloat16* xsm = bsm + SDC_Q * LDN;
        // the weighted x as three terms
        for (int i = tid; i < SDC_Q * (PT / 2); i += SDC_THREADS) {
            const int t = i / (PT / 2), p = (i % (PT / 2)) * 2;
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(xsm + t * LDP + p));
            const float w = we[t];
            uint32_t q[3];
            sd_split3(w * v.x, w * v.y, q);
#pragma unroll
            for (int k = 0; k < 3; ++k) *reinterpret_cast<uint32_t*>(xterm + (k * SDC_Q + t) * LDP + p) = q[k];
        }
        // y of the state before the chunk, and the scores C_t . B_s of the tokens up to t
        float y[YB][4], gs[8][4];
#pragma unroll
        for (int j = 0; j < YB; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; ++j) gs[j][0] = gs[j][1] = gs[j][2] = gs[j][3] = 0.0f;
        const int sblocks = tr / 16 + 1;                               // 16-token blocks s <= t
#pragma unroll 2
        for (int ks = 0; ks < NP / 16; ++ks) {
            uint32_t fa[4], fb[4];
            sd_ldm(fa, sd_smem(csm + (tr + (lmat & 1) * 8 + lrow) * LDN + ks * 16 + (lmat >> 1) * 8));
#pragma unroll
            for (int k = 0; k < 3; ++k)
#pragma unroll
                for (int j = 0; j < YB; j += 2) {
                    sd_ldm_t(fb, sd_smem(sterm + (k * NP + ks * 16 + (lmat & 1) * 8 + lrow) * LDP + yc + j * 8 + (lmat >> 1) * 8));
                    sd_mma(y[j], fa, fb[0], fb[1]);
                    sd_mma(y[j + 1], fa, fb[2], fb[3]);
                }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (j >= sblocks) continue;
                sd_ldm(fb, sd_smem(bsm + (j * 16 + (lmat >> 1) * 8 + lrow) * LDN + ks * 16 + (lmat & 1) * 8));
                sd_mma(gs[2 * j], fa, fb[0], fb[1]);
                sd_mma(gs[2 * j + 1], fa, fb[2], fb[3]);
            }
        }
        const int ta = tr + (lane >> 2), tb = ta + 8;                  // the fragment's token rows
        const float Aa = A[ta], Ab = A[tb];
        {
            const float ea = fm_ex2(Aa), eb = fm_ex2(Ab);
#pragma unroll
            for (int j = 0; j < YB; ++j) { y[j][0] *= ea; y[j][1] *= ea; y[j][2] *= eb; y[j][3] *= eb; }
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (kk >= sblocks) continue;
            uint32_t w[4][3];                                          // the fragment's four registers, three terms each
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int s = kk * 16 + half * 8 + (lane & 3) * 2;
                const float* q = gs[2 * kk + half];
                const float A0 = A[s], A1 = A[s + 1], d0 = dt[s], d1 = dt[s + 1];
                // min: the sums of later tokens may round above the earlier one's by nothing but rounding
                const float m0 = s <= ta ? q[0] * fm_ex2(fminf(Aa - A0, 0.0f)) * d0 : 0.0f, m1 = s + 1 <= ta ? q[1] * fm_ex2(fminf(Aa - A1, 0.0f)) * d1 : 0.0f;
                const float m2 = s <= tb ? q[2] * fm_ex2(fminf(Ab - A0, 0.0f)) * d0 : 0.0f, m3 = s + 1 <= tb ? q[3] * fm_ex2(fminf(Ab - A1, 0.0f)) * d1 : 0.0f;
                sd_split3(m0, m1, w[2 * half]);
                sd_split3(m2, m3, w[2 * half + 1]);
            }
#pragma unroll
            for (int j = 0; j < YB; j += 2) {
                uint32_t fb[4];
                sd_ldm_t(fb, sd_smem(xsm + (kk * 16 + (lmat & 1) * 8 + lrow) * LDP + yc + j * 8 + (lmat >> 1) * 8));
#pragma unroll
                for (int k = 0; k < 3; ++k) {
                    const uint32_t fa[4] = {w[0][k], w[1][k], w[2][k], w[3][k]};
                    sd_mma(y[j], fa, fb[0], fb[1]);
                    sd_mma(y[j + 1], fa, fb[2], fb[3]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < YB; ++j) {
            const int p = yc + j * 8 + (lane & 3) * 2;
            if (p0 + p >= a.P) continue;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int t = half ? tb : ta;
                if (t0 + t >= len) continue;
                const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(xsm + t * LDP + p));
                *reinterpret_cast<float2*>(a.y + (size_t)(row0 + t0 + t) * a.ldy + (size_t)h * a.P + p0 + p) =
                    make_float2(fmaf(dh, v.x, y[j][2 * half]), fmaf(dh, v.y, y[j][2 * half + 1]));
            }
        }
        __syncthreads();                                               // the state's terms have been read, those of the weighted x are there
        {
            const float e = fm_ex2(A[SDC_Q - 1]);
#pragma unroll
            for (int j = 0; j < SB; ++j) { S[j][0] *= e; S[j][1] *= e; S[j][2] *= e; S[j][3] *= e; }
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t fa[4];                                            // B^T: rows are state numbers, k the tokens
            sd_ldm_t(fa, sd_smem(bsm + (kk * 16 + (lmat >> 1) * 8 + lrow) * LDN + rt * 16 + (lmat & 1) * 8));
#pragma unroll
            for (int k = 0; k < 3; ++k)
#pragma unroll
                for (int j = 0; j < SB; j += 2) {
                    uint32_t fb[4];
                    sd_ldm_t(fb, sd_smem(xterm + (k * SDC_Q + kk * 16 + (lmat & 1) * 8 + lrow) * LDP + sc0 + j * 8 + (lmat >> 1) * 8));
                    sd_mma(S[j], fa, fb[0], fb[1]);
                    sd_mma(S[j + 1], fa, fb[2], fb[3]);
                }
        }
        if (t0 + SDC_Q < len) keep_terms();
    }
#pragma unroll
    for (int j = 0; j < SB; ++j) {
        const int c = p0 + sq + 8 * j;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int n = sr + 8 * half;
            if (n < a.N && c < a.P) *reinterpret_cast<float2*>(st + (size_t)n * a.P + c) = make_float2(S[j][2 * half], S[j][2 * half + 1]);
        }
    }
}

template <int NP, int PT>
static int launch_chunk(const DualArgs& a, int n_reqs, cudaStream_t s) {
    constexpr int bytes = DualShape<NP, PT>::BYTES;
    static_assert(bytes <= 227 * 1024, "fits an SM's shared memory");
    static unsigned long long configured = 0;
    if (int e = vcb_allow_dynamic_smem(state_dual_chunk_kernel<NP, PT>, bytes, &configured)) return e;
    vcb_launch(state_dual_chunk_kernel<NP, PT>, dim3((a.P + PT - 1) / PT, a.H, n_reqs), SDC_THREADS, (size_t)bytes, s, a);
    return vcb_last_error();
}

// walk 1: the walking kernel whatever the portions (both kernels compute the same).
VCB_EXPORT int vcb_state_dual(const void* x, long long ldx, const void* b, long long ldb, const void* c, long long ldc, const void* dt_pre,
                              long long lddt, const float* dt_bias, const float* a2, const float* d, float* state, float* y, long long ldy,
                              const int* q_start, const int* state_slots, int n_reqs, int max_q_len, int H, int G, int N, int P, int walk,
                              int dtype, void* stream) {
    if (n_reqs <= 0 || max_q_len <= 0) return 0;
    if (!x || !b || !c || !dt_pre || !dt_bias || !a2 || !d || !state || !y || H <= 0 || G <= 0 || H % G || N <= 0 || P <= 0 || n_reqs > 65535 || H > 65535)
        return VCB_ERR_BAD_ARG;
    if (N > 512) return VCB_ERR_UNSUPPORTED;
    DualArgs a{x, b, c, dt_pre, ldx, ldb, ldc, lddt, dt_bias, a2, d, state, y, ldy, q_start, state_slots, H, G, N, P};
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == VCB_F32) return launch_walk<float>(a, n_reqs, s);
    if (dtype != VCB_BF16) return VCB_ERR_BAD_ARG;
    const bool aligned = !((N | P) & 7) && !((ldx | ldb | ldc) & 7) && !(((uintptr_t)x | (uintptr_t)b | (uintptr_t)c) & 15) && !(ldy & 1) && !((uintptr_t)y & 7);
    if (walk || max_q_len < 16 || !aligned || N > 128) return launch_walk<__nv_bfloat16>(a, n_reqs, s);
    // narrow tiles where wide ones would leave SMs without a CTA
    const bool wide = P > 32 && (long long)n_reqs * H * ((P + 63) / 64) * 2 > vcb_sm_count();
    if (N <= 64) return wide ? launch_chunk<64, 64>(a, n_reqs, s) : launch_chunk<64, 32>(a, n_reqs, s);
    return wide ? launch_chunk<128, 64>(a, n_reqs, s) : launch_chunk<128, 32>(a, n_reqs, s);
}
