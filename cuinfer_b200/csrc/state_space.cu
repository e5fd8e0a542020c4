// The state-space recurrence with a scalar decay per head (the Mamba-2 form), and the gated norm that follows it.
//
// Rows [x (H P) | B (G N) | C (G N)] of every token, a step size per head dt = softplus(z + dt_bias), head h with the B and C of
// group h / (H / G); S is [P][N] (a head's state; N values of one output side by side):
//
//   S <- exp(-exp(A_log) dt) S + dt x B^T;     y = S C + D x
//
// Requests, slots and the order of tokens as in recurrent.cu.  Step sizes, decays, state and read-out are 32-bit.
//
// Two kernels.  A step of several requests runs both: requests of up to kSsmFewTokens tokens walk (a decoded token beside a
// prompt's portion would cost a whole chunk), longer ones go in chunks.
//  * ssm_walk: token after token in 32-bit FMA, any sizes; a warp holds four rows of S over its lanes.  Steps of single tokens,
//    the 32-bit engine, sizes the other does not take.
//  * ssm_chunk (bfloat16 rows): 64 tokens at a time on the tensor cores.  With L_t the sum of the log decays of a chunk's tokens
//    up to t, and S0 the state before the chunk,
//        y_t = exp(L_t) S0 C_t + sum_(s <= t) [exp(L_t - L_s) dt_s (C_t . B_s)] x_s + D x_t
//        S   = exp(L_end) S0 + sum_s [exp(L_end - L_s) dt_s x_s] B_s^T
//    x, B and C enter as they are stored; the 32-bit factors — S0 and the bracketed values — enter as two bfloat16 numbers
//    each (value and remainder), so that a product keeps 16 bits of them.  S0 stays in registers as the accumulators of the
//    update, whose layout is that of a product's first operand.
#include "mma_utils.cuh"
#include "scan_utils.cuh"

namespace cib {

constexpr int kSsmFewTokens = 16;
constexpr int kSsmWarps = 4, kSsmRows = 4;       // a block walks kSsmWarps * kSsmRows rows of a head's state

template <typename T, int C>
__global__ void __launch_bounds__(kSsmWarps * 32)
ssm_walk_kernel(const T* __restrict__ rows, int stride, const float* __restrict__ z, int z_stride, AnyVec dt_bias, AnyVec a_log, AnyVec skip,
                float* __restrict__ state, const int* __restrict__ query_start_loc, const int* __restrict__ state_slots, int num_slots,
                float* __restrict__ out, int H, int G, int P, int N, int few) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = blockIdx.x, h = blockIdx.y, p0 = (blockIdx.z * kSsmWarps + warp) * kSsmRows;
    griddep_launch();
    const float a = -expf(a_log[h]), bias = dt_bias[h], dskip = skip[h];          // weights
    griddep_wait();
    const int t0 = query_start_loc[r], t1 = query_start_loc[r + 1];
    if (t1 <= t0 || p0 >= P || (few > 0 && t1 - t0 > few)) return;
    const int slot = state_slots[r];
    const bool has = slot >= 0 && slot < num_slots;
    float* st = has ? state + (((size_t)slot * H + h) * P + p0) * N : nullptr;
    float S[kSsmRows][C];
#pragma unroll
    for (int q = 0; q < kSsmRows; ++q)
#pragma unroll
        for (int c = 0; c < C; ++c) S[q][c] = (has && p0 + q < P && c * 32 + lane < N) ? st[(size_t)q * N + c * 32 + lane] : 0.f;
    const T* x_ = rows + (size_t)h * P + p0;
    const T* b_ = rows + (size_t)H * P + (size_t)(h / (H / G)) * N;
    const T* c_ = b_ + (size_t)G * N;
    float nb[C], nc[C], nx[kSsmRows], nz;
    auto fetch = [&](int t) {
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const bool ok = c * 32 + lane < N;
            nb[c] = ok ? to_f32(b_[(size_t)t * stride + c * 32 + lane]) : 0.f;
            nc[c] = ok ? to_f32(c_[(size_t)t * stride + c * 32 + lane]) : 0.f;
        }
#pragma unroll
        for (int q = 0; q < kSsmRows; ++q) nx[q] = p0 + q < P ? to_f32(x_[(size_t)t * stride + q]) : 0.f;
        nz = z[(size_t)t * z_stride + h];
    };
    fetch(t0);
    for (int t = t0; t < t1; ++t) {
        float b[C], cc[C], x[kSsmRows];
#pragma unroll
        for (int c = 0; c < C; ++c) { b[c] = nb[c]; cc[c] = nc[c]; }
#pragma unroll
        for (int q = 0; q < kSsmRows; ++q) x[q] = nx[q];
        const float dt = softplusf_(nz + bias);
        if (t + 1 < t1) fetch(t + 1);                       // the next token's values are on their way meanwhile
        // g S as keep S + (g - keep) S, keep = 1 for a slow decay: what a decay close to one takes off is then rounded by
        // itself, not with the one (over a thousand tokens the difference is a digit)
        const float ld = a * dt, keep = ld > -0.5f ? 1.f : 0.f, rest = keep != 0.f ? expm1f(ld) : expf(ld);
        float y[kSsmRows];
#pragma unroll
        for (int q = 0; q < kSsmRows; ++q) {
            const float xd = dt * x[q];
            float acc = 0.f;
#pragma unroll
            for (int c = 0; c < C; ++c) {
                S[q][c] = fmaf(keep, S[q][c], fmaf(rest, S[q][c], xd * b[c]));
                acc = fmaf(S[q][c], cc[c], acc);
            }
            y[q] = acc;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int q = 0; q < kSsmRows; ++q) y[q] += __shfl_xor_sync(0xffffffffu, y[q], o);
#pragma unroll
        for (int q = 0; q < kSsmRows; ++q)
            if (lane == q && p0 + q < P) out[(size_t)t * H * P + (size_t)h * P + p0 + q] = fmaf(dskip, x[q], y[q]);
    }
    if (!has) return;
#pragma unroll
    for (int q = 0; q < kSsmRows; ++q)
#pragma unroll
        for (int c = 0; c < C; ++c)
            if (p0 + q < P && c * 32 + lane < N) st[(size_t)q * N + c * 32 + lane] = S[q][c];
}

// ---- chunks of 64 tokens on the tensor cores -----------------------------------------------------------------------------
constexpr int kChunk = 64;
constexpr int kChunkLd = kChunk + 8;
constexpr int kChunkThreads = 256;

__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(&hi);
    lo = pack_bf16(a - __low2float(h), b - __high2float(h));
}

template <int NP> constexpr int ssm_stages() { return NP <= 128 ? 3 : 2; }
template <int NP, int TILES> constexpr size_t ssm_chunk_smem() {
    constexpr int PT = TILES * 16;
    return (size_t)ssm_stages<NP>() * (2 * kChunk * (NP + 8) + kChunk * (PT + 8)) * 2      // C, B, x of a chunk
           + (size_t)2 * 2 * kChunk * (PT + 8) * 2                          // two chunks' weighted x, value and remainder
           + (size_t)2 * 2 * kChunk * kChunkLd * 2                          // two chunks' weights of pairs, likewise
           + (size_t)3 * 5 * kChunk * 4                                     // three chunks' L, dt, exp(L), weights of the update, of pairs
           + (TILES < 4 ? (size_t)4 * 8 * 32 * 16 : 0);                     // the consumers' parts of y
}

// A CTA walks the chunks of one request for 16 TILES rows of one head's S.  Only the state links one chunk to the next, so
// the warps divide: four producers make the next chunk's weighted x and pair weights (16 tokens each, and the first of them
// the step sizes of the chunk after it), four consumers take the current chunk's products with S.  One barrier a chunk.
// A consumer holds 16 rows and 1 / SPLIT of the columns of S (SPLIT = 4 / TILES: the tensor pipe of a warp's scheduler is what
// bounds a chunk's time, so a prompt with too few heads to fill the GPU shares a row tile out to several schedulers); the
// parts of y that its columns and its share of the pairs give are then added through shared memory.
template <int NP, int TILES>
__global__ void __launch_bounds__(kChunkThreads)
ssm_chunk_kernel(const __nv_bfloat16* __restrict__ rows, int stride, const float* __restrict__ z, int z_stride, AnyVec dt_bias, AnyVec a_log,
                 AnyVec skip, float* __restrict__ state, const int* __restrict__ query_start_loc, const int* __restrict__ state_slots,
                 int num_slots, float* __restrict__ out, int H, int G, int P, int N, int few) {
    constexpr int PT = TILES * 16, LDN = NP + 8, LDP = PT + 8, STAGES = ssm_stages<NP>(), SPLIT = 4 / TILES, NS = NP / SPLIT;
    static_assert(NS % 16 == 0, "a warp's columns are whole steps of a product");
    constexpr int kStage = 2 * kChunk * LDN + kChunk * LDP;
    extern __shared__ __align__(16) unsigned char ssm_raw[];
    __nv_bfloat16* stages = reinterpret_cast<__nv_bfloat16*>(ssm_raw);
    __nv_bfloat16* xw = stages + STAGES * kStage;               // [2 chunks][value, remainder][kChunk][LDP]
    __nv_bfloat16* pw = xw + 4 * kChunk * LDP;                  // [2 chunks][value, remainder][kChunk][kChunkLd]
    float* steps = reinterpret_cast<float*>(pw + 4 * kChunk * kChunkLd);      // [3 chunks][L, dt, exp(L), update, pairs][kChunk]
    float4* parts = reinterpret_cast<float4*>(steps + 3 * 5 * kChunk);        // [consumer][j][lane]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool producer = warp >= 4;
    const int r = blockIdx.z, h = blockIdx.x, p_base = blockIdx.y * PT;
    const int t0 = query_start_loc[r], t1 = query_start_loc[r + 1];
    if (t1 - t0 <= few) return;
    const int chunks = (t1 - t0 + kChunk - 1) / kChunk;
    const int slot = state_slots[r];
    const bool has = slot >= 0 && slot < num_slots;
    const int qrow = lane >> 2, quad = lane & 3, mat = lane >> 3, rr = lane & 7;
    const float a = -expf(a_log[h]), bias = dt_bias[h], dskip = skip[h];
    const __nv_bfloat16* x_ = rows + (size_t)h * P + p_base;
    const __nv_bfloat16* b_ = rows + (size_t)H * P + (size_t)(h / (H / G)) * N;
    const __nv_bfloat16* c_ = b_ + (size_t)G * N;

    auto load = [&](int c) {                                    // a token or column beyond the rows becomes zero
        const int base = t0 + c * kChunk, count = min(kChunk, t1 - base);
        __nv_bfloat16* cs = stages + (c % STAGES) * kStage;
        __nv_bfloat16 *bs = cs + kChunk * LDN, *xs = bs + kChunk * LDN;
        for (int idx = tid; idx < kChunk * (NP / 8); idx += kChunkThreads) {
            const int s = idx / (NP / 8), n = (idx % (NP / 8)) * 8;
            const bool ok = s < count && n < N;
            const size_t at = ok ? (size_t)(base + s) * stride + n : 0;
            cp_async16(cs + s * LDN + n, c_ + at, ok);
            cp_async16(bs + s * LDN + n, b_ + at, ok);
        }
        for (int idx = tid; idx < kChunk * (PT / 8); idx += kChunkThreads) {
            const int s = idx / (PT / 8), p = (idx % (PT / 8)) * 8;
            const bool ok = s < count && p_base + p < P;
            cp_async16(xs + s * LDP + p, x_ + (ok ? (size_t)(base + s) * stride + p : 0), ok);
        }
    };
    // the step sizes of a chunk, by one warp: tokens 2 lane and 2 lane + 1; a token beyond the rows has a step of zero
    auto raw_step = [&](int c, int s) {
        const int t = t0 + c * kChunk + s;
        return t < t1 ? z[(size_t)t * z_stride + h] : 0.f;
    };
    auto step_sizes = [&](int c, float z0, float z1) {
        const int count = min(kChunk, t1 - (t0 + c * kChunk));
        float* Ls = steps + (c % 3) * 5 * kChunk;
        float *dts = Ls + kChunk, *eL = dts + kChunk, *wu = eL + kChunk, *wp = wu + kChunk;
        const float d0 = 2 * lane < count ? softplusf_(z0 + bias) : 0.f, d1 = 2 * lane + 1 < count ? softplusf_(z1 + bias) : 0.f;
        const float l1 = a * d1;
        float sum = fmaf(a, d0, l1);                            // inclusive over the lanes' pairs
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += v;
        }
        const float end = __shfl_sync(0xffffffffu, sum, 31), first = sum - l1;
        *reinterpret_cast<float2*>(Ls + 2 * lane) = make_float2(first, sum);
        *reinterpret_cast<float2*>(dts + 2 * lane) = make_float2(d0, d1);
        *reinterpret_cast<float2*>(eL + 2 * lane) = make_float2(expf(first), expf(sum));
        *reinterpret_cast<float2*>(wu + 2 * lane) = make_float2(expf(end - first) * d0, expf(end - sum) * d1);
        const float edge = __shfl_sync(0xffffffffu, sum, lane | 7);          // at the last of the token's sixteen
        *reinterpret_cast<float2*>(wp + 2 * lane) = make_float2(expf(edge - first) * d0, expf(edge - sum) * d1);
    };

    load(0);
    cp_async_commit();
    if (warp == 4) step_sizes(0, raw_step(0, 2 * lane), raw_step(0, 2 * lane + 1));
    const int tile = warp % TILES, share = (warp / TILES) % SPLIT, n_base = share * NS;      // a consumer's rows and columns
    const int p_lo = p_base + tile * 16 + qrow, p_hi = p_lo + 8;
    const bool mine = !producer && p_base + tile * 16 < P;
    float S[NS / 8][4];                                          // rows p_lo, p_hi; columns n_base + 8 j + 2 quad, + 1
    if (mine) {
        const float* st = has ? state + ((size_t)slot * H + h) * P * N : nullptr;
#pragma unroll
        for (int j = 0; j < NS / 8; ++j) {
            const int n = n_base + j * 8 + quad * 2;
            const float2 lo = has && n < N && p_lo < P ? *reinterpret_cast<const float2*>(st + (size_t)p_lo * N + n) : make_float2(0.f, 0.f);
            const float2 hi = has && n < N && p_hi < P ? *reinterpret_cast<const float2*>(st + (size_t)p_hi * N + n) : make_float2(0.f, 0.f);
            S[j][0] = lo.x; S[j][1] = lo.y; S[j][2] = hi.x; S[j][3] = hi.y;
        }
    }
    for (int c = -1; c < chunks; ++c) {                          // producers are one chunk ahead
        cp_async_wait<0>();                                      // this thread's copies of chunk c + 1
        __syncthreads();                                         // everyone's, and everyone is done with chunk c - 1
        if (STAGES == 3 && c + 2 < chunks) load(c + 2);
        if (STAGES == 2 && c == -1 && chunks > 1) load(1);
        cp_async_commit();
        if (producer) {
            if (c + 1 < chunks) {
                const int pc = c + 1, w4 = warp - 4, ptid = tid - 128;
                const bool ahead = w4 == 0 && pc + 1 < chunks;
                float z0 = 0.f, z1 = 0.f;
                if (ahead) {
                    z0 = raw_step(pc + 1, 2 * lane);
                    z1 = raw_step(pc + 1, 2 * lane + 1);
                }
                const __nv_bfloat16* cs = stages + (pc % STAGES) * kStage;
                const __nv_bfloat16 *bs = cs + kChunk * LDN, *xs = bs + kChunk * LDN;
                const float* Ls = steps + (pc % 3) * 5 * kChunk;
                const float *dts = Ls + kChunk, *wu = Ls + 3 * kChunk, *wp = Ls + 4 * kChunk;
                __nv_bfloat16 *xw_hi = xw + (pc & 1) * 2 * kChunk * LDP, *xw_lo = xw_hi + kChunk * LDP;
                __nv_bfloat16 *w_hi = pw + (pc & 1) * 2 * kChunk * kChunkLd, *w_lo = w_hi + kChunk * kChunkLd;
#pragma unroll 4
                for (int idx = ptid; idx < kChunk * (PT / 4); idx += 128) {
                    const int s = idx / (PT / 4), p = (idx % (PT / 4)) * 4;
                    const uint2 v = *reinterpret_cast<const uint2*>(xs + s * LDP + p);
                    const float2 v0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
                    const float2 v1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
                    const float f = wu[s];
                    uint2 hi, lo;
                    split_bf16(f * v0.x, f * v0.y, hi.x, lo.x);
                    split_bf16(f * v1.x, f * v1.y, hi.y, lo.y);
                    *reinterpret_cast<uint2*>(xw_hi + s * LDP + p) = hi;
                    *reinterpret_cast<uint2*>(xw_lo + s * LDP + p) = lo;
                }
                // this warp's rows of C B^T, weighted; tiles above the diagonal are never read
                const int tr = w4 * 16;
                float g[kChunk / 8][4];
#pragma unroll
                for (int j = 0; j < kChunk / 8; ++j) g[j][0] = g[j][1] = g[j][2] = g[j][3] = 0.f;
#pragma unroll 4
                for (int kk = 0; kk < NP / 16; ++kk) {
                    uint32_t af[4];
                    ldmatrix_x4(af, smem_u32(cs + (tr + (mat & 1) * 8 + rr) * LDN + kk * 16 + (mat >> 1) * 8));
#pragma unroll
                    for (int np = 0; np < kChunk / 16; ++np) {
                        if (np > w4) continue;
                        uint32_t bf[4];
                        ldmatrix_x4(bf, smem_u32(bs + (np * 16 + (mat >> 1) * 8 + rr) * LDN + kk * 16 + (mat & 1) * 8));
                        mma_bf16_16816(g[2 * np], af, bf[0], bf[1]);
                        mma_bf16_16816(g[2 * np + 1], af, bf[2], bf[3]);
                    }
                }
                const int ta = tr + qrow, tb = ta + 8;
                // exp(L_t - L_s) of tokens in different sixteens goes by way of the earlier sixteen's last token, whose L lies
                // between the two: one factor a token and sixteen instead of one a pair, neither above one
                const float La = Ls[ta], Lb = Ls[tb];
#pragma unroll
                for (int np = 0; np < kChunk / 16; ++np) {
                    if (np > w4) continue;
                    const float edge = Ls[np * 16 + 15];
                    const bool diagonal = np == w4;
                    const float fa = diagonal ? 1.f : expf(La - edge), fb = diagonal ? 1.f : expf(Lb - edge);
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        const int j = 2 * np + half, s = j * 8 + quad * 2;
                        float2 va, vb;
                        if (diagonal) {
                            const float2 ls = *reinterpret_cast<const float2*>(Ls + s), d = *reinterpret_cast<const float2*>(dts + s);
                            va = make_float2(s <= ta ? expf(La - ls.x) * d.x : 0.f, s + 1 <= ta ? expf(La - ls.y) * d.y : 0.f);
                            vb = make_float2(s <= tb ? expf(Lb - ls.x) * d.x : 0.f, s + 1 <= tb ? expf(Lb - ls.y) * d.y : 0.f);
                        } else {
                            const float2 w = *reinterpret_cast<const float2*>(wp + s);
                            va = make_float2(fa * w.x, fa * w.y);
                            vb = make_float2(fb * w.x, fb * w.y);
                        }
                        uint32_t hi, lo;
                        split_bf16(g[j][0] * va.x, g[j][1] * va.y, hi, lo);
                        *reinterpret_cast<uint32_t*>(w_hi + ta * kChunkLd + s) = hi;
                        *reinterpret_cast<uint32_t*>(w_lo + ta * kChunkLd + s) = lo;
                        split_bf16(g[j][2] * vb.x, g[j][3] * vb.y, hi, lo);
                        *reinterpret_cast<uint32_t*>(w_hi + tb * kChunkLd + s) = hi;
                        *reinterpret_cast<uint32_t*>(w_lo + tb * kChunkLd + s) = lo;
                    }
                }
                if (ahead) step_sizes(pc + 1, z0, z1);
            }
        } else if (c >= 0) {
            const __nv_bfloat16* cs = stages + (c % STAGES) * kStage;
            const __nv_bfloat16 *bs = cs + kChunk * LDN, *xs = bs + kChunk * LDN;
            const float* eL = steps + (c % 3) * 5 * kChunk + 2 * kChunk;
            const __nv_bfloat16 *xw_hi = xw + (c & 1) * 2 * kChunk * LDP, *xw_lo = xw_hi + kChunk * LDP;
            const __nv_bfloat16 *w_hi = pw + (c & 1) * 2 * kChunk * kChunkLd, *w_lo = w_hi + kChunk * kChunkLd;
            // y = S0 C^T: rows of S from the registers
            float y[kChunk / 8][4];
#pragma unroll
            for (int j = 0; j < kChunk / 8; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
            if (mine) {
#pragma unroll
                for (int kk = 0; kk < NS / 16; ++kk) {
                    uint32_t hi[4], lo[4];
                    split_bf16(S[2 * kk][0], S[2 * kk][1], hi[0], lo[0]);
                    split_bf16(S[2 * kk][2], S[2 * kk][3], hi[1], lo[1]);
                    split_bf16(S[2 * kk + 1][0], S[2 * kk + 1][1], hi[2], lo[2]);
                    split_bf16(S[2 * kk + 1][2], S[2 * kk + 1][3], hi[3], lo[3]);
                    uint32_t bf[kChunk / 16][4];
#pragma unroll
                    for (int np = 0; np < kChunk / 16; ++np)
                        ldmatrix_x4(bf[np], smem_u32(cs + (np * 16 + (mat >> 1) * 8 + rr) * LDN + n_base + kk * 16 + (mat & 1) * 8));
#pragma unroll
                    for (int np = 0; np < kChunk / 16; ++np) {
                        mma_bf16_16816(y[2 * np], hi, bf[np][0], bf[np][1]);
                        mma_bf16_16816(y[2 * np + 1], hi, bf[np][2], bf[np][3]);
                    }
#pragma unroll
                    for (int np = 0; np < kChunk / 16; ++np) {
                        mma_bf16_16816(y[2 * np], lo, bf[np][0], bf[np][1]);
                        mma_bf16_16816(y[2 * np + 1], lo, bf[np][2], bf[np][3]);
                    }
                }
#pragma unroll
                for (int j = 0; j < kChunk / 8; ++j) {
                    const float2 e = *reinterpret_cast<const float2*>(eL + j * 8 + quad * 2);
                    y[j][0] *= e.x; y[j][1] *= e.y; y[j][2] *= e.x; y[j][3] *= e.y;
                }
                const float e_end = eL[kChunk - 1];
#pragma unroll
                for (int j = 0; j < NS / 8; ++j) { S[j][0] *= e_end; S[j][1] *= e_end; S[j][2] *= e_end; S[j][3] *= e_end; }
#pragma unroll
                for (int kk = 0; kk < kChunk / 16; ++kk) {
                    const int s0 = kk * 16;
                    uint32_t xa[4], wa_hi[4], wa_lo[4];
                    const int at = (s0 + (mat >> 1) * 8 + rr) * LDP + tile * 16 + (mat & 1) * 8;
                    ldmatrix_x4_trans(wa_hi, smem_u32(xw_hi + at));
                    ldmatrix_x4_trans(wa_lo, smem_u32(xw_lo + at));
                    const bool pairs_here = kk % SPLIT == share;     // this consumer's share of the chunk's own pairs
                    if (pairs_here) ldmatrix_x4_trans(xa, smem_u32(xs + at));
#pragma unroll
                    for (int np = 0; np < kChunk / 16; ++np) {
                        if (np < kk || !pairs_here) continue;        // tokens before s0 do not see it
                        uint32_t bh[4], bl[4];
                        ldmatrix_x4(bh, smem_u32(w_hi + (np * 16 + (mat >> 1) * 8 + rr) * kChunkLd + s0 + (mat & 1) * 8));
                        ldmatrix_x4(bl, smem_u32(w_lo + (np * 16 + (mat >> 1) * 8 + rr) * kChunkLd + s0 + (mat & 1) * 8));
                        mma_bf16_16816(y[2 * np], xa, bh[0], bh[1]);
                        mma_bf16_16816(y[2 * np + 1], xa, bh[2], bh[3]);
                        mma_bf16_16816(y[2 * np], xa, bl[0], bl[1]);
                        mma_bf16_16816(y[2 * np + 1], xa, bl[2], bl[3]);
                    }
#pragma unroll
                    for (int nj = 0; nj < NS / 16; ++nj) {
                        uint32_t bf[4];
                        ldmatrix_x4_trans(bf, smem_u32(bs + (s0 + (mat & 1) * 8 + rr) * LDN + n_base + nj * 16 + (mat >> 1) * 8));
                        mma_bf16_16816(S[2 * nj], wa_hi, bf[0], bf[1]);
                        mma_bf16_16816(S[2 * nj + 1], wa_hi, bf[2], bf[3]);
                        mma_bf16_16816(S[2 * nj], wa_lo, bf[0], bf[1]);
                        mma_bf16_16816(S[2 * nj + 1], wa_lo, bf[2], bf[3]);
                    }
                }
            }
            if constexpr (SPLIT > 1) {                           // the consumers of a row tile add up: each for its share of the tokens
#pragma unroll
                for (int j = 0; j < kChunk / 8; ++j) parts[(warp * 8 + j) * 32 + lane] = make_float4(y[j][0], y[j][1], y[j][2], y[j][3]);
                asm volatile("bar.sync 1, 128;" ::: "memory");   // the four consumer warps
#pragma unroll
                for (int i = 0; i < kChunk / 8 / SPLIT; ++i) {
                    const int j = share * (kChunk / 8 / SPLIT) + i;
                    float4 sum = parts[(tile * 8 + j) * 32 + lane];
#pragma unroll
                    for (int o = 1; o < SPLIT; ++o) {
                        const float4 v = parts[((tile + o * TILES) * 8 + j) * 32 + lane];
                        sum.x += v.x; sum.y += v.y; sum.z += v.z; sum.w += v.w;
                    }
                    y[i][0] = sum.x; y[i][1] = sum.y; y[i][2] = sum.z; y[i][3] = sum.w;
                }
            }
            const int base = t0 + c * kChunk, count = mine ? min(kChunk, t1 - base) : 0;
            const int xl = tile * 16 + qrow;                     // this lane's rows within x's columns
#pragma unroll
            for (int i = 0; i < kChunk / 8 / SPLIT; ++i) {
                const int j = share * (kChunk / 8 / SPLIT) + i;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int s = j * 8 + quad * 2 + e;
                    if (s >= count) continue;
                    float* dst = out + ((size_t)(base + s) * H + h) * P;
                    if (p_lo < P) dst[p_lo] = fmaf(dskip, __bfloat162float(xs[s * LDP + xl]), y[i][e]);
                    if (p_hi < P) dst[p_hi] = fmaf(dskip, __bfloat162float(xs[s * LDP + xl + 8]), y[i][2 + e]);
                }
            }
        }
        if (STAGES == 2 && c >= 0 && c + 2 < chunks) {           // the stage of chunk c is free only now
            __syncthreads();
            load(c + 2);
            cp_async_commit();
        }
    }
    if (!has || !mine) return;
    float* st = state + ((size_t)slot * H + h) * P * N;
#pragma unroll
    for (int j = 0; j < NS / 8; ++j) {
        const int n = n_base + j * 8 + quad * 2;
        if (n >= N) continue;
        if (p_lo < P) *reinterpret_cast<float2*>(st + (size_t)p_lo * N + n) = make_float2(S[j][0], S[j][1]);
        if (p_hi < P) *reinterpret_cast<float2*>(st + (size_t)p_hi * N + n) = make_float2(S[j][2], S[j][3]);
    }
}

// ---- the gate, then an RMS norm in groups, then the gain --------------------------------------------------------------------
// v = y * silu(z);  out = v / sqrt(mean over the group of v^2 + eps) * gain.  A block per (token, group), v in shared memory.
template <typename TZ, typename TO, int V>
__global__ void __launch_bounds__(256)
gated_group_rms_kernel(const float* __restrict__ y, const TZ* __restrict__ z, int z_stride, AnyVec gain, float eps, TO* __restrict__ out,
                       int groups, int width) {
    extern __shared__ __align__(16) float gated_s[];
    __shared__ float scratch[33];
    griddep_launch();
    griddep_wait();
    const int t = blockIdx.x / groups, g = blockIdx.x % groups;
    const size_t at = (size_t)blockIdx.x * width;
    const TZ* zr = z + (size_t)t * z_stride + (size_t)g * width;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float v[V], zz[V];
        if constexpr (V == 4) {
            const float4 f = *reinterpret_cast<const float4*>(y + at + i);
            v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
            if constexpr (sizeof(TZ) == 2) {
                const uint2 u = *reinterpret_cast<const uint2*>(zr + i);
                const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&u.x), b = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
                zz[0] = __low2float(a); zz[1] = __high2float(a); zz[2] = __low2float(b); zz[3] = __high2float(b);
            } else {
                const float4 f2 = *reinterpret_cast<const float4*>(zr + i);
                zz[0] = f2.x; zz[1] = f2.y; zz[2] = f2.z; zz[3] = f2.w;
            }
        } else {
            v[0] = y[at + i];
            zz[0] = to_f32(zr[i]);
        }
#pragma unroll
        for (int k = 0; k < V; ++k) {
            v[k] *= zz[k] / (1.f + expf(-zz[k]));
            ss = fmaf(v[k], v[k], ss);
            gated_s[i + k] = v[k];
        }
    }
    ss = block_sum(ss, scratch);
    const float factor = 1.f / sqrtf(ss / (float)width + eps);
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {           // the elements this thread has written itself
        float v[V];
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = gated_s[i + k] * factor * gain[g * width + i + k];
        if constexpr (V == 4 && sizeof(TO) == 2) *reinterpret_cast<uint2*>(out + at + i) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
        else if constexpr (V == 4) *reinterpret_cast<float4*>(out + at + i) = make_float4(v[0], v[1], v[2], v[3]);
        else out[at + i] = from_f32<TO>(v[0]);
    }
}

}  // namespace cib

using namespace cib;

extern "C" int cib_ssm_chunk_supports(int H, int G, int P, int N) {
    return H > 0 && G > 0 && P % 8 == 0 && N % 8 == 0 && N <= 256 && H % G == 0;
}

template <int NP, int TILES>
static int launch_ssm_chunk_tiles(const void* rows, int stride, const float* z, int z_stride, AnyVec db, AnyVec al, AnyVec sk, float* state,
                            const int* query_start_loc, const int* state_slots, int num_slots, int num_requests, float* out, int H, int G, int P,
                            int N, int few, cudaStream_t stream) {
    constexpr size_t smem = ssm_chunk_smem<NP, TILES>();
    static_assert(smem <= 227 * 1024, "a chunk's working set does not fit");
    static SmemLimit limit;
    if (int rc = raise_smem_limit(limit, ssm_chunk_kernel<NP, TILES>, smem, "ssm_chunk")) return rc;
    const dim3 grid(H, (P + TILES * 16 - 1) / (TILES * 16), num_requests);
    ssm_chunk_kernel<NP, TILES><<<grid, kChunkThreads, smem, stream>>>((const __nv_bfloat16*)rows, stride, z, z_stride, db, al, sk, state, query_start_loc,
                                                               state_slots, num_slots, out, H, G, P, N, few);
    CIB_LAUNCH_CHECK("ssm_chunk");
    return 0;
}

// Row tiles a CTA: as few as leave every CTA an SM of its own.
template <int NP>
static int launch_ssm_chunk(const void* rows, int stride, const float* z, int z_stride, AnyVec db, AnyVec al, AnyVec sk, float* state,
                            const int* query_start_loc, const int* state_slots, int num_slots, int num_requests, float* out, int H, int G, int P,
                            int N, int few, cudaStream_t stream) {
    auto ctas = [&](int tiles) { return (long long)num_requests * H * ((P + tiles * 16 - 1) / (tiles * 16)); };
#define CIB_SSM_TILES(TILES)                                                                                                             \
    return launch_ssm_chunk_tiles<NP, TILES>(rows, stride, z, z_stride, db, al, sk, state, query_start_loc, state_slots, num_slots,          \
                                             num_requests, out, H, G, P, N, few, stream)
    if constexpr (NP >= 64)
        if (ctas(1) <= 148) CIB_SSM_TILES(1);
    if (ctas(2) <= 148) CIB_SSM_TILES(2);
    CIB_SSM_TILES(4);
#undef CIB_SSM_TILES
}

// rows [tokens][>= H P + 2 G N] `stride` apart; z float32 step-size logits [tokens][>= H] `z_stride` apart; dt_bias, a_log, skip [H];
// state float32 [slots][H][P][N]; out float32 [tokens][H P].  chunks: take the tensor-core form (bfloat16 rows on 16-byte
// boundaries, sizes in multiples of 8).
extern "C" int cib_ssm_scan(const void* rows, int dtype, int stride, const float* z, int z_stride, const void* dt_bias, const void* a_log,
                            const void* skip, int vec_dtype, float* state, const int* query_start_loc, const int* state_slots, int num_slots,
                            int num_requests, int num_tokens, float* out, int H, int G, int P, int N, int chunks, cudaStream_t stream) {
    CIB_REQUIRE(H > 0 && G > 0 && H % G == 0 && P > 0 && N > 0 && stride >= H * P + 2 * G * N && z_stride >= H, "ssm_scan: bad sizes");
    CIB_REQUIRE(N <= 256, "ssm_scan: state size %d is beyond 256", N);
    if (num_requests == 0 || num_tokens == 0) return 0;
    AnyVec db{dt_bias, vec_dtype == kBF16}, al{a_log, vec_dtype == kBF16}, sk{skip, vec_dtype == kBF16};
    const int few = chunks && num_requests > 1 ? kSsmFewTokens : 0;
    if (chunks) {
        CIB_REQUIRE(dtype == kBF16 && cib_ssm_chunk_supports(H, G, P, N) && stride % 8 == 0 && (uintptr_t)rows % 16 == 0 && (uintptr_t)state % 16 == 0,
                    "ssm_scan: the rows do not fit the tensor-core form");
        CIB_REQUIRE(num_requests <= 65535, "ssm_scan: too many requests");
        int rc;
#define CIB_SSM(NP)                                                                                                                       \
    rc = launch_ssm_chunk<NP>(rows, stride, z, z_stride, db, al, sk, state, query_start_loc, state_slots, num_slots, num_requests, out, H, G, P, \
                              N, few, stream)
        if (N <= 32) CIB_SSM(32);
        else if (N <= 64) CIB_SSM(64);
        else if (N <= 128) CIB_SSM(128);
        else CIB_SSM(256);
#undef CIB_SSM
        if (rc != 0 || few == 0) return rc;
    }
    const dim3 grid(num_requests, H, (P + kSsmWarps * kSsmRows - 1) / (kSsmWarps * kSsmRows));
    const bool pdl = prompt_pdl();
#define CIB_WALK(T, C)                                                                                                                    \
    launch_pdl(ssm_walk_kernel<T, C>, grid, dim3(kSsmWarps * 32), 0, stream, pdl, (const T*)rows, stride, z, z_stride, db, al, sk, state,      \
               query_start_loc, state_slots, num_slots, out, H, G, P, N, few)
#define CIB_WALK_N(T)                         \
    do {                                      \
        if (N <= 32) CIB_WALK(T, 1);          \
        else if (N <= 64) CIB_WALK(T, 2);     \
        else if (N <= 128) CIB_WALK(T, 4);    \
        else CIB_WALK(T, 8);                  \
    } while (0)
    if (dtype == kF32) CIB_WALK_N(float);
    else if (dtype == kBF16) CIB_WALK_N(__nv_bfloat16);
    else CIB_REQUIRE(false, "ssm_scan: bad dtype %d", dtype);
#undef CIB_WALK_N
#undef CIB_WALK
    CIB_LAUNCH_CHECK("ssm_scan");
    return 0;
}

// y float32 [tokens][groups * width]; z rows `z_stride` apart; gain [groups * width]; out [tokens][groups * width].
extern "C" int cib_gated_group_rms(const float* y, const void* z, int z_dtype, int z_stride, const void* gain, int gain_dtype, float eps,
                                   void* out, int out_dtype, int groups, int width, int num_tokens, cudaStream_t stream) {
    CIB_REQUIRE(groups > 0 && width > 0 && z_stride >= groups * width && num_tokens >= 0, "gated_group_rms: bad sizes");
    CIB_REQUIRE(width <= 12 * 1024, "gated_group_rms: groups of %d values are beyond this kernel", width);
    CIB_REQUIRE((long long)num_tokens * groups < (1ll << 31), "gated_group_rms: too many rows");
    if (num_tokens == 0) return 0;
    AnyVec gv{gain, gain_dtype == kBF16};
    const bool v4 = width % 4 == 0 && z_stride % 4 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)z % (z_dtype == kF32 ? 16 : 8) == 0 &&
                    (uintptr_t)out % 16 == 0;
    int threads = 32;
    while (threads < 256 && threads * (v4 ? 4 : 1) < width) threads <<= 1;
    const size_t smem = (size_t)width * sizeof(float);
    const bool pdl = prompt_pdl();
#define CIB_GATED(TZ, TO, V)                                                                                                            \
    launch_pdl(gated_group_rms_kernel<TZ, TO, V>, dim3((unsigned)(num_tokens * groups)), dim3(threads), smem, stream, pdl, y, (const TZ*)z,   \
               z_stride, gv, eps, (TO*)out, groups, width)
    if (z_dtype == kF32 && out_dtype == kF32) { if (v4) CIB_GATED(float, float, 4); else CIB_GATED(float, float, 1); }
    else if (z_dtype == kF32 && out_dtype == kBF16) { if (v4) CIB_GATED(float, __nv_bfloat16, 4); else CIB_GATED(float, __nv_bfloat16, 1); }
    else if (z_dtype == kBF16 && out_dtype == kBF16) { if (v4) CIB_GATED(__nv_bfloat16, __nv_bfloat16, 4); else CIB_GATED(__nv_bfloat16, __nv_bfloat16, 1); }
    else CIB_REQUIRE(false, "gated_group_rms: bad dtypes %d -> %d", z_dtype, out_dtype);
#undef CIB_GATED
    CIB_LAUNCH_CHECK("gated_group_rms");
    return 0;
}
