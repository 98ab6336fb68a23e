// Paged attention over a sliding window of tokens and, for what lies before the window, one mean key and one mean value per
// block of P tokens; queries, keys and values pass a short causal convolution, queries and keys a rotation first:
//
//   conv_rope_cache_write_kernel   bias, convolution over time (state in the request's slot), rotation of interleaved pairs,
//                                  a factor per query head; keys and values into the token's slot of the cache, queries out
//   pool_blocks_kernel             the blocks of P tokens that this step completes: the mean of their keys and of their values
//                                  as the cache holds them, into the block's row of a second group of pages (a row per block)
//   attention_pooled_kernel        softmax over both: the query at position i sees the tokens j with 0 <= i - j < W and the
//                                  blocks b with (b + 1) P - 1 <= i - W; the plain form (a warp per token and head, a key per
//                                  lane), both storage types.  W = 0: every token, no blocks.  P = 0: no blocks.
//
// Both groups' pages have the layout of kv_pos (common.cuh) with rows of max(dk, dv) elements.  Angles, convolution, means,
// scores, softmax and sums are float.  The reference's attention (src/attention/paged_attention.cu) has none of this.
#include "short_conv.cuh"

struct ConvRopeArgs {
    const void* proj;           // [n, ...] rows that hold a token's q, k and v projections one after the other
    long long ld;
    const float* bias;          // [C] or null: added in the projection; C = nh * dk + nkv * (dk + dv)
    const float* taps;          // [C, J]
    float* state;               // slot s, row j, channel c at state[s * slot_stride + j * C + c]
    long long slot_stride;
    const float* inv_freq;      // [rot / 2] or null
    const float* q_factor;      // [nh] or null: multiplies a head's queries
    void* q_out;                // [n, nh * dk]
    void* cache;
    const int* q_start;
    const int* positions;
    const int* state_slots;
    const int* block_table;
    int bt_stride, nh, nkv, dk, dv, row, page, num_pages, rot, J;
    int* status;
};

// Grid (segments of the longest portion, requests, tiles of 128 pairs of channels): a thread per pair of neighbouring
// channels of a head (the pairs the rotation turns) and segment of SEG tokens.  VEC: head sizes, offsets and strides are even,
// so a pair is one access.  J <= MAXJ.
template <typename T, int MAXJ, int SEG, bool VEC>
__global__ void __launch_bounds__(128) conv_rope_cache_write_kernel(ConvRopeArgs a) {
    const int pq = (a.dk + 1) >> 1, pv = (a.dv + 1) >> 1;
    const int nq = a.nh * pq, nk = a.nkv * pq, total = nq + nk + a.nkv * pv;
    const int p = blockIdx.z * 128 + threadIdx.x;
    const bool there = p < total;
    const int kind = p < nq ? 0 : p < nq + nk ? 1 : 2;             // q, k, v
    const int at = kind == 0 ? p : kind == 1 ? p - nq : p - nq - nk;
    const int per = kind == 2 ? pv : pq, dim = kind == 2 ? a.dv : a.dk;
    const int head = at / per, i = at - head * per;
    const int live = min(2, dim - 2 * i);
    const int C = a.nh * a.dk + a.nkv * (a.dk + a.dv);
    const int c = (kind == 0 ? 0 : kind == 1 ? a.nh * a.dk : (a.nh + a.nkv) * a.dk) + head * dim + 2 * i;
    float taps[MAXJ][2], pb[2] = {0.0f, 0.0f};
    float factor = 1.0f, freq = 0.0f;
    if (there) {
        conv_taps<MAXJ, 2>(a.taps + (size_t)c * a.J, a.J, live, taps);
        if (a.bias) {
            pb[0] = a.bias[c];
            if (live == 2) pb[1] = a.bias[c + 1];
        }
        if (kind == 0 && a.q_factor) factor = a.q_factor[head];
        if (kind < 2 && 2 * i < a.rot) freq = a.inv_freq[i];
    }
    const bool turns = kind < 2 && 2 * i < a.rot;
    pdl_start();
    const int r = blockIdx.y;
    const int row0 = a.q_start[r], len = a.q_start[r + 1] - row0;
    const int seg0 = blockIdx.x * SEG;
    if (seg0 >= len || !there) return;
    const int pos0 = a.positions[row0];
    const T* x = (const T*)a.proj + (size_t)row0 * a.ld + c;
    float* st = a.state + (size_t)a.state_slots[r] * a.slot_stride + c;
    float h[MAXJ - 1 + SEG][2];
    if (VEC) conv_window<T, MAXJ, SEG, 2>(x, a.ld, st, C, pb, a.J, seg0, len, 2, h);
    else {
        // pairs that may lie on odd addresses: an element at a time
        float h0[MAXJ - 1 + SEG][1], h1[MAXJ - 1 + SEG][1];
        const float b0[1] = {pb[0]}, b1[1] = {pb[1]};
        conv_window<T, MAXJ, SEG, 1>(x, a.ld, st, C, b0, a.J, seg0, len, 1, h0);
        if (live == 2) conv_window<T, MAXJ, SEG, 1>(x + 1, a.ld, st + 1, C, b1, a.J, seg0, len, 1, h1);
#pragma unroll
        for (int k = 0; k < MAXJ - 1 + SEG; ++k) { h[k][0] = h0[k][0]; h[k][1] = live == 2 ? h1[k][0] : 0.0f; }
    }
    const size_t block = (size_t)a.page * a.row, page_elems = 2 * (size_t)a.nkv * block;
    const int* bt = a.block_table + (size_t)r * a.bt_stride;
    bool bad = false;
#pragma unroll
    for (int t = 0; t < SEG; ++t) {
        const int li = seg0 + t;
        if (li >= len) break;
        float y0 = 0.0f, y1 = 0.0f;
#pragma unroll
        for (int m = 0; m < MAXJ; ++m) { y0 = fmaf(taps[m][0], h[t + m][0], y0); y1 = fmaf(taps[m][1], h[t + m][1], y1); }
        const int pos = pos0 + li;
        if (turns) {
            float sn, cs;
            sincosf((float)pos * freq, &sn, &cs);
            const float u = y0, v = y1;
            y0 = u * cs - v * sn;
            y1 = v * cs + u * sn;
        }
        T* dst;
        if (kind == 0) {
            dst = (T*)a.q_out + (size_t)(row0 + li) * a.nh * a.dk + head * a.dk + 2 * i;
            y0 *= factor;
            y1 *= factor;
        } else {
            const int lp = pos / a.page, slot = pos - lp * a.page;
            const int pg = lp < a.bt_stride ? bt[lp] : -1;
            if ((unsigned)pg >= (unsigned)a.num_pages) { bad = true; continue; }
            // a pair never leaves its 16-byte chunk
            dst = (T*)a.cache + (size_t)pg * page_elems + (size_t)(kind == 1 ? head : a.nkv + head) * block
                  + kv_pos(2 * i, slot, a.row, a.page, (int)sizeof(T));
        }
        if (VEC && sizeof(T) == 2) {
            *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(y0, y1);
        } else if (VEC) {
            *reinterpret_cast<float2*>(dst) = make_float2(y0, y1);
        } else {
            dst[0] = from_f32<T>(y0);
            if (live == 2) dst[1] = from_f32<T>(y1);
        }
    }
    if (bad && a.status) atomicCAS(a.status, 0, VCB_STATUS_BAD_PAGE);
    if (seg0 == 0) conv_keep<T, 2>(x, a.ld, st, C, pb, a.J, len, live);
}

// Any number of taps up to POOLED_LONG_TAPS, read from memory one by one; segments as long as the taps allow.
#define POOLED_LONG_TAPS 64
template <typename T>
__global__ void __launch_bounds__(128) conv_rope_cache_write_long_kernel(ConvRopeArgs a) {
    constexpr int SEG = POOLED_LONG_TAPS;
    const int pq = (a.dk + 1) >> 1, pv = (a.dv + 1) >> 1;
    const int nq = a.nh * pq, nk = a.nkv * pq, total = nq + nk + a.nkv * pv;
    const int p = blockIdx.z * 128 + threadIdx.x;
    pdl_start();
    const int r = blockIdx.y;
    const int row0 = a.q_start[r], len = a.q_start[r + 1] - row0;
    const int seg0 = blockIdx.x * SEG;
    if (seg0 >= len || p >= total) return;
    const int kind = p < nq ? 0 : p < nq + nk ? 1 : 2;
    const int at = kind == 0 ? p : kind == 1 ? p - nq : p - nq - nk;
    const int per = kind == 2 ? pv : pq, dim = kind == 2 ? a.dv : a.dk;
    const int head = at / per, i = at - head * per;
    const int live = min(2, dim - 2 * i);
    const int C = a.nh * a.dk + a.nkv * (a.dk + a.dv);
    const int c = (kind == 0 ? 0 : kind == 1 ? a.nh * a.dk : (a.nh + a.nkv) * a.dk) + head * dim + 2 * i;
    const int pos0 = a.positions[row0];
    const T* x = (const T*)a.proj + (size_t)row0 * a.ld + c;
    float* st = a.state + (size_t)a.state_slots[r] * a.slot_stride + c;
    float pb[2] = {0.0f, 0.0f};
    if (a.bias) for (int e = 0; e < live; ++e) pb[e] = a.bias[c + e];
    const size_t block = (size_t)a.page * a.row, page_elems = 2 * (size_t)a.nkv * block;
    const int* bt = a.block_table + (size_t)r * a.bt_stride;
    for (int li = seg0; li < min(seg0 + SEG, len); ++li) {
        float y[2] = {0.0f, 0.0f};
        for (int j = 0; j < a.J; ++j) {
            const int s = li - (a.J - 1) + j;
            for (int e = 0; e < live; ++e) {
                const float u = s >= 0 ? to_f32<T>(x[(size_t)s * a.ld + e]) + pb[e] : st[(size_t)(a.J - 1 + s) * C + e];
                y[e] = fmaf(a.taps[(size_t)(c + e) * a.J + j], u, y[e]);
            }
        }
        const int pos = pos0 + li;
        if (kind < 2 && 2 * i < a.rot) {
            float sn, cs;
            sincosf((float)pos * a.inv_freq[i], &sn, &cs);
            const float u = y[0], v = y[1];
            y[0] = u * cs - v * sn;
            y[1] = v * cs + u * sn;
        }
        T* dst;
        if (kind == 0) {
            dst = (T*)a.q_out + (size_t)(row0 + li) * a.nh * a.dk + head * a.dk + 2 * i;
            if (a.q_factor) for (int e = 0; e < 2; ++e) y[e] *= a.q_factor[head];
        } else {
            const int lp = pos / a.page, slot = pos - lp * a.page;
            const int pg = lp < a.bt_stride ? bt[lp] : -1;
            if ((unsigned)pg >= (unsigned)a.num_pages) {
                if (a.status) atomicCAS(a.status, 0, VCB_STATUS_BAD_PAGE);
                continue;
            }
            dst = (T*)a.cache + (size_t)pg * page_elems + (size_t)(kind == 1 ? head : a.nkv + head) * block
                  + kv_pos(2 * i, slot, a.row, a.page, (int)sizeof(T));
        }
        for (int e = 0; e < live; ++e) dst[e] = from_f32<T>(y[e]);
    }
    if (seg0 == 0) conv_keep<T, 2>(x, a.ld, st, C, pb, a.J, len, live);
}

template <typename T, int MAXJ, int SEG>
static void launch_conv_rope(const ConvRopeArgs& a, int n_reqs, int max_q_len, int pairs, bool vec, cudaStream_t s) {
    dim3 grid((max_q_len + SEG - 1) / SEG, n_reqs, (pairs + 127) / 128);
    if (vec) vcb_launch(conv_rope_cache_write_kernel<T, MAXJ, SEG, true>, grid, 128, 0, s, a);
    else vcb_launch(conv_rope_cache_write_kernel<T, MAXJ, SEG, false>, grid, 128, 0, s, a);
}

template <typename T>
static int launch_conv_rope_any(const ConvRopeArgs& a, int n_reqs, int max_q_len, cudaStream_t s) {
    const int pairs = (a.nh + a.nkv) * ((a.dk + 1) / 2) + a.nkv * ((a.dv + 1) / 2);
    const uintptr_t addrs = (uintptr_t)a.proj | (uintptr_t)a.q_out | (uintptr_t)a.cache;
    const bool vec = !((a.dk | a.dv | a.row) & 1) && !(a.ld & 1) && !(addrs & (2 * sizeof(T) - 1));
    if (a.J > 8) {
        dim3 grid((max_q_len + POOLED_LONG_TAPS - 1) / POOLED_LONG_TAPS, n_reqs, (pairs + 127) / 128);
        vcb_launch(conv_rope_cache_write_long_kernel<T>, grid, 128, 0, s, a);
    } else if (max_q_len == 1) {
        if (a.J <= 4) launch_conv_rope<T, 4, 1>(a, n_reqs, 1, pairs, vec, s);
        else launch_conv_rope<T, 8, 1>(a, n_reqs, 1, pairs, vec, s);
    } else {
        if (a.J <= 4) launch_conv_rope<T, 4, 16>(a, n_reqs, max_q_len, pairs, vec, s);
        else launch_conv_rope<T, 8, 16>(a, n_reqs, max_q_len, pairs, vec, s);
    }
    return vcb_last_error();
}

VCB_EXPORT int vcb_conv_rope_cache_write(const void* proj, long long ld, const float* bias, const float* taps, int J, float* state,
                                         long long slot_stride, const float* inv_freq, int rot, const float* q_factor, void* q_out,
                                         void* cache, const int* q_start, const int* positions, const int* state_slots,
                                         const int* block_table, int bt_stride, int n_reqs, int max_q_len, int nh, int nkv, int dk,
                                         int dv, int row, int page, int num_pages, int* status, int dtype, void* stream) {
    if (n_reqs <= 0 || max_q_len <= 0) return 0;
    if (!proj || !taps || !state || !q_out || !cache || nh <= 0 || nkv <= 0 || dk <= 0 || dv <= 0 || row < dk || row < dv || page <= 0 ||
        J < 1 || J > POOLED_LONG_TAPS || rot < 0 || rot > dk || (rot & 1) || (rot && !inv_freq) || n_reqs > 65535)
        return VCB_ERR_BAD_ARG;
    ConvRopeArgs a{proj, ld, bias, taps, state, slot_stride, inv_freq, q_factor, q_out, cache, q_start, positions, state_slots, block_table,
                   bt_stride, nh, nkv, dk, dv, row, page, num_pages, rot, J, status};
    if (dtype == VCB_F32) return launch_conv_rope_any<float>(a, n_reqs, max_q_len, (cudaStream_t)stream);
    if (dtype == VCB_BF16) return launch_conv_rope_any<__nv_bfloat16>(a, n_reqs, max_q_len, (cudaStream_t)stream);
    return VCB_ERR_BAD_ARG;
}

// ---------------------------------------------------------------------------------------- block means
struct PoolArgs {
    const void* cache;          // pages of tokens
    void* pooled;               // pages of blocks
    const int* q_start;
    const int* ctx_lens;
    const int* block_table;     // of the tokens' group
    const int* pool_table;      // of the blocks' group
    int bt_stride, pt_stride, nkv, dk, dv, row, page, num_pages, pool_pages, P;
    int* status;
};

// Grid (blocks a request can complete in this step, requests, kv heads): block ctx / P + blockIdx.x of the request, if this
// step brings its last token.  Keys and then values; a thread per VW neighbouring elements, the block's tokens in order.
template <typename T, int VW>
__global__ void __launch_bounds__(128) pool_blocks_kernel(PoolArgs a) {
    pdl_start();
    const int r = blockIdx.y, g = blockIdx.z;
    const int ctx = a.ctx_lens[r], len = a.q_start[r + 1] - a.q_start[r];
    const int b = ctx / a.P + blockIdx.x;
    if ((b + 1) * a.P > ctx + len) return;
    const int* bt = a.block_table + (size_t)r * a.bt_stride;
    const int prow = b / a.page, pslot = b - prow * a.page;
    const int ppg = prow < a.pt_stride ? a.pool_table[(size_t)r * a.pt_stride + prow] : -1;
    const size_t block = (size_t)a.page * a.row, page_elems = 2 * (size_t)a.nkv * block;
    if ((unsigned)ppg >= (unsigned)a.pool_pages) {
        if (a.status && threadIdx.x == 0) atomicCAS(a.status, 0, VCB_STATUS_BAD_PAGE);
        return;
    }
    const int first = b * a.P, lp0 = first / a.page, slot0 = first - lp0 * a.page;
    for (int e = threadIdx.x * VW; e < a.dk + a.dv; e += blockDim.x * VW) {
        const bool is_v = e >= a.dk;
        const int el = is_v ? e - a.dk : e;
        const size_t head = (size_t)(is_v ? a.nkv + g : g) * block;
        float sum[VW];
#pragma unroll
        for (int i = 0; i < VW; ++i) sum[i] = 0.0f;
#pragma unroll 8
        for (int k = 0; k < a.P; ++k) {
            const int at = slot0 + k, over = at / a.page, slot = at - over * a.page, lp = lp0 + over;
            const int pg = lp < a.bt_stride ? bt[lp] : -1;
            if ((unsigned)pg >= (unsigned)a.num_pages) {
                if (a.status) atomicCAS(a.status, 0, VCB_STATUS_BAD_PAGE);
                continue;
            }
            float v[VW];
            conv_load<T, VW>((const T*)a.cache + (size_t)pg * page_elems + head + kv_pos(el, slot, a.row, a.page, (int)sizeof(T)), v);
#pragma unroll
            for (int i = 0; i < VW; ++i) sum[i] += v[i];
        }
        T* dst = (T*)a.pooled + (size_t)ppg * page_elems + head + kv_pos(el, pslot, a.row, a.page, (int)sizeof(T));
#pragma unroll
        for (int i = 0; i < VW; ++i) dst[i] = from_f32<T>(sum[i] / (float)a.P);
    }
}

VCB_EXPORT int vcb_pool_blocks(const void* cache, void* pooled, const int* q_start, const int* ctx_lens, const int* block_table,
                               int bt_stride, const int* pool_table, int pt_stride, int n_reqs, int max_q_len, int nkv, int dk, int dv,
                               int row, int page, int num_pages, int pool_pages, int P, int* status, int dtype, void* stream) {
    if (n_reqs <= 0 || max_q_len <= 0) return 0;
    if (!cache || !pooled || nkv <= 0 || dk <= 0 || dv <= 0 || row < dk || row < dv || page <= 0 || P <= 0 || n_reqs > 65535 || nkv > 65535)
        return VCB_ERR_BAD_ARG;
    PoolArgs a{cache, pooled, q_start, ctx_lens, block_table, pool_table, bt_stride, pt_stride, nkv, dk, dv, row, page, num_pages, pool_pages,
               P, status};
    // a portion of n tokens completes at most ceil(n / P) blocks
    dim3 grid((max_q_len + P - 1) / P, n_reqs, nkv);
    cudaStream_t s = (cudaStream_t)stream;
    const bool pairs = !((dk | dv | row) & 1) && !(((uintptr_t)cache | (uintptr_t)pooled) & 7);
    if (dtype == VCB_F32 && pairs) vcb_launch(pool_blocks_kernel<float, 2>, grid, 128, 0, s, a);
    else if (dtype == VCB_F32) vcb_launch(pool_blocks_kernel<float, 1>, grid, 128, 0, s, a);
    else if (dtype == VCB_BF16 && pairs) vcb_launch(pool_blocks_kernel<__nv_bfloat16, 2>, grid, 128, 0, s, a);
    else if (dtype == VCB_BF16) vcb_launch(pool_blocks_kernel<__nv_bfloat16, 1>, grid, 128, 0, s, a);
    else return VCB_ERR_BAD_ARG;
    return vcb_last_error();
}

// ---------------------------------------------------------------------------------------- attention, plain form
#define APL_MAX_DV 512
#define APL_WARPS 4

struct PooledAttnArgs {
    const void* q;              // [n, nh * dk]
    const void* cache;          // pages of tokens
    const void* pooled;         // pages of blocks (null: P = 0)
    void* out;                  // [n, nh * dv]
    const int* positions;
    const int* req_of_token;
    const int* block_table;
    const int* pool_table;
    int bt_stride, pt_stride, n_tokens, nh, nkv, dk, dv, row, page, window, P, num_pages, pool_pages;
    float scale;
    int* status;
};

template <typename T, int MAXDV>
__global__ void attention_pooled_kernel(PooledAttnArgs a) {
    extern __shared__ float qs_all[];
    pdl_start();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * APL_WARPS + warp;
    if (item >= (long long)a.n_tokens * a.nh) return;
    const int t = (int)(item / a.nh), h = (int)(item % a.nh);
    const int g = h / (a.nh / a.nkv);
    const int pos = a.positions[t], r = a.req_of_token[t];
    float* qs = qs_all + warp * a.dk;
    const T* qrow = (const T*)a.q + ((size_t)t * a.nh + h) * a.dk;
    for (int i = lane; i < a.dk; i += 32) qs[i] = to_f32<T>(qrow[i]);
    __syncwarp();

    const size_t block = (size_t)a.page * a.row;
    const size_t page_elems = 2 * (size_t)a.nkv * block, v_off = (size_t)a.nkv * block;
    float o[MAXDV / 32];
#pragma unroll
    for (int k = 0; k < MAXDV / 32; ++k) o[k] = 0.0f;
    float m = -INFINITY, l = 0.0f;

    // the same walk over blocks (0 .. blocks - 1) and then over tokens (first .. pos)
    const int first = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    const int blocks = (a.window > 0 && a.P > 0) ? first / a.P : 0;
    for (int part = blocks > 0 ? 0 : 1; part < 2; ++part) {
        const T* cache = (const T*)(part == 0 ? a.pooled : a.cache);
        const int* bt = part == 0 ? a.pool_table + (size_t)r * a.pt_stride : a.block_table + (size_t)r * a.bt_stride;
        const int stride = part == 0 ? a.pt_stride : a.bt_stride, pages = part == 0 ? a.pool_pages : a.num_pages;
        const int lo = part == 0 ? 0 : first, hi = part == 0 ? blocks : pos + 1;
        for (int kb = lo; kb < hi; kb += 32) {
            const int j = kb + lane;
            bool valid = j < hi;
            float s = -INFINITY;
            unsigned long long koff = 0;
            if (valid) {
                const int lp = j / a.page;
                const int pg = lp < stride ? bt[lp] : -1;
                if ((unsigned)pg >= (unsigned)pages) {
                    if (a.status) atomicCAS(a.status, 0, VCB_STATUS_BAD_PAGE);
                    valid = false;
                } else {
                    koff = (unsigned long long)pg * page_elems + (size_t)g * block;
                }
            }
            if (valid) {
                const T* kr = cache + koff;
                const int slot = j % a.page;
                float acc = 0.0f;
                for (int i = 0; i < a.dk; ++i) acc += qs[i] * to_f32<T>(kr[kv_pos(i, slot, a.row, a.page, (int)sizeof(T))]);
                s = acc * a.scale;
            }
            const float m_new = fmaxf(m, warp_max(s));
            const float corr = m_new == -INFINITY ? 1.0f : expf(m - m_new);
            const float p = valid ? expf(s - m_new) : 0.0f;
            l = l * corr + warp_sum(p);
#pragma unroll
            for (int k = 0; k < MAXDV / 32; ++k) o[k] *= corr;
            const int nvalid = min(32, hi - kb);
            for (int jj = 0; jj < nvalid; ++jj) {
                const float pj = __shfl_sync(0xffffffffu, p, jj);
                const unsigned long long off = __shfl_sync(0xffffffffu, koff, jj);
                const T* vr = cache + off + v_off;
                const int slot = (kb + jj) % a.page;
#pragma unroll
                for (int k = 0; k < MAXDV / 32; ++k) {
                    const int dim = lane + 32 * k;
                    if (dim < a.dv) o[k] += pj * to_f32<T>(vr[kv_pos(dim, slot, a.row, a.page, (int)sizeof(T))]);
                }
            }
            m = m_new;
        }
    }
    T* orow = (T*)a.out + ((size_t)t * a.nh + h) * a.dv;
    const float inv = l > 0.0f ? 1.0f / l : 0.0f;
#pragma unroll
    for (int k = 0; k < MAXDV / 32; ++k) {
        const int dim = lane + 32 * k;
        if (dim < a.dv) orow[dim] = from_f32<T>(o[k] * inv);
    }
}

template <typename T>
static int launch_pooled(const PooledAttnArgs& a, cudaStream_t s) {
    const long long items = (long long)a.n_tokens * a.nh;
    const int blocks = (int)((items + APL_WARPS - 1) / APL_WARPS);
    const size_t smem = (size_t)APL_WARPS * a.dk * sizeof(float);
    if (a.dv <= 128) vcb_launch(attention_pooled_kernel<T, 128>, blocks, APL_WARPS * 32, smem, s, a);
    else vcb_launch(attention_pooled_kernel<T, APL_MAX_DV>, blocks, APL_WARPS * 32, smem, s, a);
    return vcb_last_error();
}

VCB_EXPORT int vcb_attention_pooled(const void* q, const void* cache, const void* pooled, void* out, const int* positions,
                                    const int* req_of_token, const int* block_table, int bt_stride, const int* pool_table, int pt_stride,
                                    int n_tokens, int nh, int nkv, int dk, int dv, int row, int page, int window, int P, float scale,
                                    int num_pages, int pool_pages, int* status, int dtype, void* stream) {
    if (n_tokens <= 0) return 0;
    if (!q || !cache || !out || dk <= 0 || dv <= 0 || dv > APL_MAX_DV || dk > 1024 || row < dk || row < dv || nh <= 0 || nkv <= 0 ||
        nh % nkv || page <= 0 || window < 0 || P < 0 || num_pages < 0 || (P > 0 && window > 0 && (!pooled || !pool_table)))
        return VCB_ERR_BAD_ARG;
    PooledAttnArgs a{q, cache, pooled, out, positions, req_of_token, block_table, pool_table, bt_stride, pt_stride, n_tokens, nh, nkv, dk, dv,
                     row, page, window, P, num_pages, pool_pages, scale, status};
    if (dtype == VCB_F32) return launch_pooled<float>(a, (cudaStream_t)stream);
    if (dtype == VCB_BF16) return launch_pooled<__nv_bfloat16>(a, (cudaStream_t)stream);
    return VCB_ERR_BAD_ARG;
}
