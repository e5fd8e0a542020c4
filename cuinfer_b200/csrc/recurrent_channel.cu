// Recurrences whose decay is a vector: every key channel (row of a head's matrix) fades at a rate of its own per token.
// The gated delta rule in that form, and the time mixing of the RWKV family with its token shift and its bonus for the
// current token.  Layout of requests, slots and columns as in recurrent.cu; everything here is 32-bit.
//
// Per head, decay g (one number per row of S):
//   delta: S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   wkv:   o = (S + diag(b) k v^T)^T r;  S <- diag(g) S + k v^T          (b: the bonus, a number per head and channel)
// Column j of S depends on nothing but itself, the token's rows and v_j.
//
// Two forms of each scan.  Steps of single tokens: one launch that takes the gates while it stages the token (a request's
// state is read and written once, nothing repeats).  Other steps: a first launch computes, for all tokens and heads at
// once, what does not depend on the state — decays, beta, the products k.q and b k.r — into 32-bit rows; the scan then walks
// the tokens with the rows of the next chunk on their way to shared memory (cp.async, two stages) meanwhile.
#include <type_traits>

#include "mma_utils.cuh"
#include "scan_utils.cuh"

namespace cib {

template <int DP> constexpr int channel_chunk() { return DP > 128 ? 8 : 16; }        // tokens staged at a time (48 KB)

// One token of a column segment; kq: k.q of the whole head.  Returns o of the column (every lane of the column has it).
template <int SPLIT>
__device__ __forceinline__ float delta_token(float (&S)[32], const float* kseg, const float* qseg, const float* gseg, float beta,
                                             float v, float kq) {
    float rk4[4] = {0.f, 0.f, 0.f, 0.f}, pq4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(kseg + i);
        const float4 q4 = *reinterpret_cast<const float4*>(qseg + i);
        const float4 g4 = *reinterpret_cast<const float4*>(gseg + i);
        S[i] *= g4.x;
        S[i + 1] *= g4.y;
        S[i + 2] *= g4.z;
        S[i + 3] *= g4.w;
        rk4[0] = fmaf(S[i], k4.x, rk4[0]);
        rk4[1] = fmaf(S[i + 1], k4.y, rk4[1]);
        rk4[2] = fmaf(S[i + 2], k4.z, rk4[2]);
        rk4[3] = fmaf(S[i + 3], k4.w, rk4[3]);
        pq4[0] = fmaf(S[i], q4.x, pq4[0]);
        pq4[1] = fmaf(S[i + 1], q4.y, pq4[1]);
        pq4[2] = fmaf(S[i + 2], q4.z, pq4[2]);
        pq4[3] = fmaf(S[i + 3], q4.w, pq4[3]);
    }
    const float rk = split_sum<SPLIT>((rk4[0] + rk4[1]) + (rk4[2] + rk4[3]));
    const float pq = split_sum<SPLIT>((pq4[0] + pq4[1]) + (pq4[2] + pq4[3]));
    const float u = beta * (v - rk);
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(kseg + i);
        S[i] = fmaf(k4.x, u, S[i]);
        S[i + 1] = fmaf(k4.y, u, S[i + 1]);
        S[i + 2] = fmaf(k4.z, u, S[i + 2]);
        S[i + 3] = fmaf(k4.w, u, S[i + 3]);
    }
    return pq + u * kq;
}

// now: sum_i b_i k_i r_i of the whole head.
template <int SPLIT>
__device__ __forceinline__ float wkv_token(float (&S)[32], const float* kseg, const float* rseg, const float* gseg, float v, float now) {
    float o4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(kseg + i);
        const float4 r4 = *reinterpret_cast<const float4*>(rseg + i);
        const float4 g4 = *reinterpret_cast<const float4*>(gseg + i);
        o4[0] = fmaf(S[i], r4.x, o4[0]);
        o4[1] = fmaf(S[i + 1], r4.y, o4[1]);
        o4[2] = fmaf(S[i + 2], r4.z, o4[2]);
        o4[3] = fmaf(S[i + 3], r4.w, o4[3]);
        S[i] = fmaf(g4.x, S[i], k4.x * v);
        S[i + 1] = fmaf(g4.y, S[i + 1], k4.y * v);
        S[i + 2] = fmaf(g4.z, S[i + 2], k4.z * v);
        S[i + 3] = fmaf(g4.w, S[i + 3], k4.w * v);
    }
    return fmaf(now, v, split_sum<SPLIT>((o4[0] + o4[1]) + (o4[2] + o4[3])));
}

// beta = sigmoid(zb), decay = exp(-exp(A_log) softplus(za + dt_bias)) are taken while the tokens are staged.
template <int DP>
__global__ void __launch_bounds__(kScanWarps * 32)
channel_delta_scan_kernel(const float* __restrict__ qkv, int qkv_stride, int G, const float* __restrict__ zb, int zb_stride,
                          const float* __restrict__ za, int za_stride, AnyVec a_log, AnyVec dt_bias, float* __restrict__ state,
                          const int* __restrict__ query_start_loc, const int* __restrict__ state_slots, int num_slots,
                          float* __restrict__ out, int H, int d, int dv) {
    constexpr int SPLIT = DP / 32, CPW = 32 / SPLIT, COLS = CPW * kScanWarps, CH = channel_chunk<DP>();
    __shared__ __align__(16) float ksm[CH][padded_len<DP>()];
    __shared__ __align__(16) float qsm[CH][padded_len<DP>()];
    __shared__ __align__(16) float gsm[CH][padded_len<DP>()];
    __shared__ float vsm[CH][COLS];
    __shared__ float bsm[CH];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = blockIdx.x, h = blockIdx.y;
    const int col0 = blockIdx.z * COLS;
    const int cb = warp * CPW + lane / SPLIT;
    const int j = col0 + cb, part = lane % SPLIT, i0 = part * 32;
    const bool col = j < dv;
    griddep_launch();
    griddep_wait();
    const int t0 = query_start_loc[r], t1 = query_start_loc[r + 1];
    if (t1 <= t0) return;
    const int slot = state_slots[r];
    const bool has = slot >= 0 && slot < num_slots;
    float* st = has ? state + ((size_t)slot * H + h) * d * dv : nullptr;
    float S[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) S[i] = (has && col && i0 + i < d) ? st[(size_t)(i0 + i) * dv + j] : 0.f;
    const int g_head = h / (H / G);
    const float* q = qkv + (size_t)g_head * d;
    const float* k = qkv + (size_t)(G + g_head) * d;
    const float* v = qkv + (size_t)2 * G * d + (size_t)h * dv;
    const float a = expf(a_log[h]);
    for (int base = t0; base < t1; base += CH) {
        const int count = min(CH, t1 - base);
        __syncthreads();
        for (int idx = threadIdx.x; idx < CH * DP; idx += blockDim.x) {
            const int tt = idx / DP, i = idx % DP;
            const bool ok = tt < count && i < d;
            const size_t row = (size_t)(base + tt);
            ksm[tt][pad32(i)] = ok ? k[row * qkv_stride + i] : 0.f;
            qsm[tt][pad32(i)] = ok ? q[row * qkv_stride + i] : 0.f;
            gsm[tt][pad32(i)] = ok ? expf(-a * softplusf_(za[row * za_stride + (size_t)h * d + i] + dt_bias[h * d + i])) : 0.f;
        }
        for (int idx = threadIdx.x; idx < CH * COLS; idx += blockDim.x) {
            const int tt = idx / COLS, c = idx % COLS;
            vsm[tt][c] = (tt < count && col0 + c < dv) ? v[(size_t)(base + tt) * qkv_stride + col0 + c] : 0.f;
        }
        if (threadIdx.x < CH) bsm[threadIdx.x] = threadIdx.x < count ? sigmoidf_(zb[(size_t)(base + threadIdx.x) * zb_stride + h]) : 0.f;
        __syncthreads();
        for (int tt = 0; tt < count; ++tt) {
            float kq = 0.f;
#pragma unroll
            for (int c = 0; c < SPLIT; ++c) kq = fmaf(ksm[tt][c * 36 + lane], qsm[tt][c * 36 + lane], kq);
            kq = warp_sum(kq);
            const float o = delta_token<SPLIT>(S, &ksm[tt][part * 36], &qsm[tt][part * 36], &gsm[tt][part * 36], bsm[tt], vsm[tt][cb], kq);
            if (col && part == 0) out[(size_t)(base + tt) * H * dv + (size_t)h * dv + j] = o;
        }
    }
    if (has && col) {
#pragma unroll
        for (int i = 0; i < 32; ++i)
            if (i0 + i < d) st[(size_t)(i0 + i) * dv + j] = S[i];
    }
}

// decay = exp(-exp(zw + w0)) is taken while the tokens are staged; r, k, v are rows of the engine's type.
template <typename T, int DP>
__global__ void __launch_bounds__(kScanWarps * 32)
wkv_scan_kernel(const T* __restrict__ r_, const T* __restrict__ k_, const T* __restrict__ v_, int stride,
                const float* __restrict__ zw, int zw_stride, AnyVec w0, AnyVec bonus, float* __restrict__ state,
                const int* __restrict__ query_start_loc, const int* __restrict__ state_slots, int num_slots,
                float* __restrict__ out, int H, int d, int dv) {
    constexpr int SPLIT = DP / 32, CPW = 32 / SPLIT, COLS = CPW * kScanWarps, CH = channel_chunk<DP>();
    __shared__ __align__(16) float ksm[CH][padded_len<DP>()];
    __shared__ __align__(16) float rsm[CH][padded_len<DP>()];
    __shared__ __align__(16) float gsm[CH][padded_len<DP>()];
    __shared__ float vsm[CH][COLS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = blockIdx.x, h = blockIdx.y;
    const int col0 = blockIdx.z * COLS;
    const int cb = warp * CPW + lane / SPLIT;
    const int j = col0 + cb, part = lane % SPLIT, i0 = part * 32;
    const bool col = j < dv;
    griddep_launch();
    float b[SPLIT];                                          // the bonus of this lane's channels c * 32 + lane: a weight
#pragma unroll
    for (int c = 0; c < SPLIT; ++c) b[c] = c * 32 + lane < d ? bonus[h * d + c * 32 + lane] : 0.f;
    griddep_wait();
    const int t0 = query_start_loc[r], t1 = query_start_loc[r + 1];
    if (t1 <= t0) return;
    const int slot = state_slots[r];
    const bool has = slot >= 0 && slot < num_slots;
    float* st = has ? state + ((size_t)slot * H + h) * d * dv : nullptr;
    float S[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) S[i] = (has && col && i0 + i < d) ? st[(size_t)(i0 + i) * dv + j] : 0.f;
    for (int base = t0; base < t1; base += CH) {
        const int count = min(CH, t1 - base);
        __syncthreads();
        for (int idx = threadIdx.x; idx < CH * DP; idx += blockDim.x) {
            const int tt = idx / DP, i = idx % DP;
            const bool ok = tt < count && i < d;
            const size_t at = (size_t)(base + tt) * stride + (size_t)h * d + i;
            ksm[tt][pad32(i)] = ok ? to_f32(k_[at]) : 0.f;
            rsm[tt][pad32(i)] = ok ? to_f32(r_[at]) : 0.f;
            gsm[tt][pad32(i)] = ok ? expf(-expf(zw[(size_t)(base + tt) * zw_stride + (size_t)h * d + i] + w0[h * d + i])) : 0.f;
        }
        for (int idx = threadIdx.x; idx < CH * COLS; idx += blockDim.x) {
            const int tt = idx / COLS, c = idx % COLS;
            vsm[tt][c] = (tt < count && col0 + c < dv) ? to_f32(v_[(size_t)(base + tt) * stride + (size_t)h * dv + col0 + c]) : 0.f;
        }
        __syncthreads();
        for (int tt = 0; tt < count; ++tt) {
            float now = 0.f;                                 // sum_i b_i k_i r_i
#pragma unroll
            for (int c = 0; c < SPLIT; ++c) now = fmaf(b[c] * ksm[tt][c * 36 + lane], rsm[tt][c * 36 + lane], now);
            now = warp_sum(now);
            const float o = wkv_token<SPLIT>(S, &ksm[tt][part * 36], &rsm[tt][part * 36], &gsm[tt][part * 36], vsm[tt][cb], now);
            if (col && part == 0) out[(size_t)(base + tt) * H * dv + (size_t)h * dv + j] = o;
        }
    }
    if (has && col) {
#pragma unroll
        for (int i = 0; i < 32; ++i)
            if (i0 + i < d) st[(size_t)(i0 + i) * dv + j] = S[i];
    }
}

// ---- steps that are not all single tokens -------------------------------------------------------------------------------
// A warp per (token, head): what the delta scan needs of a token beside its rows.
//   decay[t, h, :] = exp(-exp(A_log_h) softplus(za + dt_bias));  pairs[t, h] = (sigmoid(zb), k.q)
constexpr int kGatherWarps = 8;
__global__ void __launch_bounds__(kGatherWarps * 32)
channel_delta_gates_kernel(const float* __restrict__ qkv, int qkv_stride, int G, const float* __restrict__ zb, int zb_stride,
                           const float* __restrict__ za, int za_stride, AnyVec a_log, AnyVec dt_bias, float* __restrict__ decay,
                           float* __restrict__ pairs, int H, int d, long long total) {
    griddep_launch();
    griddep_wait();
    const int lane = threadIdx.x & 31;
    const long long w = (long long)blockIdx.x * kGatherWarps + (threadIdx.x >> 5);
    if (w >= total) return;
    const long long t = w / H;
    const int h = (int)(w % H), g = h / (H / G);
    const float* q = qkv + t * qkv_stride + (size_t)g * d;
    const float* k = q + (size_t)G * d;
    const float a = expf(a_log[h]);
    float kq = 0.f;
    for (int i0 = 0; i0 < d; i0 += 32) {
        const int i = i0 + lane;
        if (i >= d) continue;
        kq = fmaf(k[i], q[i], kq);
        decay[(size_t)t * H * d + (size_t)h * d + i] = expf(-a * softplusf_(za[t * za_stride + (size_t)h * d + i] + dt_bias[h * d + i]));
    }
    kq = warp_sum(kq);
    if (lane == 0) {
        pairs[w * 2] = sigmoidf_(zb[t * zb_stride + h]);
        pairs[w * 2 + 1] = kq;
    }
}

// The same for the time mixing: rows[t] = [r (H d) | k (H d) | decay (H d) | v (H dv)] in 32 bits, pairs[t, h] = (sum b k r, 0).
template <typename T>
__global__ void __launch_bounds__(kGatherWarps * 32)
wkv_rows_kernel(const T* __restrict__ r, const T* __restrict__ k, const T* __restrict__ v, int stride, const float* __restrict__ zw,
                int zw_stride, AnyVec w0, AnyVec bonus, float* __restrict__ rows, float* __restrict__ pairs, int H, int d, int dv,
                long long total) {
    griddep_launch();
    griddep_wait();
    const int lane = threadIdx.x & 31;
    const long long w = (long long)blockIdx.x * kGatherWarps + (threadIdx.x >> 5);
    if (w >= total) return;
    const long long t = w / H;
    const int h = (int)(w % H);
    float* row = rows + (size_t)t * H * (3 * d + dv);
    float now = 0.f;
    for (int i0 = 0; i0 < d; i0 += 32) {
        const int i = i0 + lane;
        if (i >= d) continue;
        const size_t at = (size_t)t * stride + (size_t)h * d + i;
        const float rv = to_f32(r[at]), kv = to_f32(k[at]);
        now = fmaf(bonus[h * d + i] * kv, rv, now);
        row[h * d + i] = rv;
        row[(size_t)H * d + h * d + i] = kv;
        row[(size_t)2 * H * d + h * d + i] = expf(-expf(zw[t * zw_stride + (size_t)h * d + i] + w0[h * d + i]));
    }
    for (int i = lane; i < dv; i += 32) row[(size_t)3 * H * d + (size_t)h * dv + i] = to_f32(v[(size_t)t * stride + (size_t)h * dv + i]);
    now = warp_sum(now);
    if (lane == 0) {
        pairs[w * 2] = now;
        pairs[w * 2 + 1] = 0.f;
    }
}

// 4- or 16-byte asynchronous copies; the staging rows are padded, so 16 bytes want sizes and strides in multiples of four.
__device__ __forceinline__ void cp_async4(float* smem, const float* gmem) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(smem_u32(smem)), "l"(gmem));
}

// The walk over the tokens.  A column of S is held by SPLIT = DP / VPL neighbouring lanes, VPL values each, dealt out four
// at a time: lane `part` holds the values (c SPLIT + part) 4 + e, so that the lanes of a column read consecutive 16 bytes of a
// staged row.  Few values a lane (8) make a token's chain of dependent operations short, which is what counts while the
// heads and columns do not fill the GPU; more (16, 32) make fewer instructions a token when they do.
// x (queries or receptances), k, g (decays), v: 32-bit rows whose strides are given; pairs: two numbers per (token, head).
constexpr long long kChannelFewWarps = 1184, kChannelManyWarps = 4736;
template <int VPL> constexpr int channel_warps() { return VPL == 8 ? 4 : 8; }
template <int DP> constexpr int channel_stage_tokens() { return DP > 128 ? 16 : 32; }

template <int VPL>
struct TokenRows {              // a lane's share of one token's rows
    float4 x[VPL / 4], k[VPL / 4], g[VPL / 4];
    template <int SPLIT>
    __device__ __forceinline__ void read(const float* xs, const float* ks, const float* gs, int part) {
#pragma unroll
        for (int c = 0; c < VPL / 4; ++c) {
            const int at = (c * SPLIT + part) * 4;
            g[c] = *reinterpret_cast<const float4*>(gs + at);
            k[c] = *reinterpret_cast<const float4*>(ks + at);
            x[c] = *reinterpret_cast<const float4*>(xs + at);
        }
    }
};
__device__ __forceinline__ float dot4(const float* s, const float4& a, float acc) {
    acc = fmaf(s[0], a.x, acc);
    acc = fmaf(s[1], a.y, acc);
    acc = fmaf(s[2], a.z, acc);
    return fmaf(s[3], a.w, acc);
}
template <int N>
__device__ __forceinline__ float sum_of(const float (&a)[N]) {       // pairwise
    float b[N];
#pragma unroll
    for (int i = 0; i < N; ++i) b[i] = a[i];
#pragma unroll
    for (int o = N / 2; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < o; ++i) b[i] += b[i + o];
    return b[0];
}

template <int DP, int VPL, bool WKV>
__global__ void __launch_bounds__(channel_warps<VPL>() * 32)
channel_scan_kernel(const float* __restrict__ x_, const float* __restrict__ k_, int xk_stride, const float* __restrict__ g_, int g_stride,
                    const float* __restrict__ v_, int v_stride, const float* __restrict__ pairs, int heads_per_key, int vec4,
                    int vec4_v, float* __restrict__ state, const int* __restrict__ query_start_loc,
                    const int* __restrict__ state_slots, int num_slots, float* __restrict__ out, int H, int d, int dv) {
    constexpr int SPLIT = DP / VPL, CPW = 32 / SPLIT, COLS = CPW * channel_warps<VPL>(), CH = channel_stage_tokens<DP>();
    constexpr int kStage = 3 * CH * DP + CH * COLS + CH * 2;
    extern __shared__ __align__(16) float smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = blockIdx.x, h = blockIdx.y;
    const int col0 = blockIdx.z * COLS;
    const int cb = warp * CPW + lane / SPLIT;
    const int j = col0 + cb, part = lane % SPLIT;
    const bool col = j < dv;
    // what no copy ever writes (values from d and dv on) stays zero
    for (int i = threadIdx.x; i < 2 * kStage; i += blockDim.x) smem[i] = 0.f;
    const int t0 = query_start_loc[r], t1 = query_start_loc[r + 1];
    if (t1 <= t0) return;
    const int slot = state_slots[r];
    const bool has = slot >= 0 && slot < num_slots;
    float* st = has ? state + ((size_t)slot * H + h) * d * dv : nullptr;
    const float* x = x_ + (size_t)(h / heads_per_key) * d;
    const float* k = k_ + (size_t)(h / heads_per_key) * d;
    const float* g = g_ + (size_t)h * d;
    const float* v = v_ + (size_t)h * dv + col0;
    const int cols = min(COLS, dv - col0);
    auto load = [&](int stage, int base, int count) {
        float* xs = smem + (size_t)stage * kStage;
        float *ks = xs + CH * DP, *gs = ks + CH * DP, *vs = gs + CH * DP, *ps = vs + CH * COLS;
        if (vec4) {
            for (int idx = threadIdx.x; idx < count * (DP / 4); idx += blockDim.x) {
                const int tt = idx / (DP / 4), i = (idx % (DP / 4)) * 4;
                if (i >= d) continue;
                const size_t t = (size_t)(base + tt);
                cp_async16(xs + tt * DP + i, x + t * xk_stride + i, true);
                cp_async16(ks + tt * DP + i, k + t * xk_stride + i, true);
                cp_async16(gs + tt * DP + i, g + t * g_stride + i, true);
            }
        } else {
            for (int idx = threadIdx.x; idx < count * DP; idx += blockDim.x) {
                const int tt = idx / DP, i = idx % DP;
                if (i >= d) continue;
                const size_t t = (size_t)(base + tt);
                cp_async4(xs + tt * DP + i, x + t * xk_stride + i);
                cp_async4(ks + tt * DP + i, k + t * xk_stride + i);
                cp_async4(gs + tt * DP + i, g + t * g_stride + i);
            }
        }
        if (vec4_v) {
            for (int idx = threadIdx.x; idx < count * (COLS / 4); idx += blockDim.x) {
                const int tt = idx / (COLS / 4), c = (idx % (COLS / 4)) * 4;
                if (c < cols) cp_async16(vs + tt * COLS + c, v + (size_t)(base + tt) * v_stride + c, true);
            }
        } else {
            for (int idx = threadIdx.x; idx < count * COLS; idx += blockDim.x) {
                const int tt = idx / COLS, c = idx % COLS;
                if (c < cols) cp_async4(vs + tt * COLS + c, v + (size_t)(base + tt) * v_stride + c);
            }
        }
        for (int idx = threadIdx.x; idx < 2 * count; idx += blockDim.x)
            cp_async4(ps + idx, pairs + ((size_t)(base + (idx >> 1)) * H + h) * 2 + (idx & 1));
    };
    __syncthreads();                                         // the zeros are in place before the first copies land
    load(0, t0, min(CH, t1 - t0));
    cp_async_commit();
    float S[VPL];
#pragma unroll
    for (int i = 0; i < VPL; ++i) {
        const int row = ((i / 4) * SPLIT + part) * 4 + i % 4;
        S[i] = (has && col && row < d) ? st[(size_t)row * dv + j] : 0.f;
    }
    int stage = 0;
    for (int base = t0; base < t1; base += CH, stage ^= 1) {
        const int count = min(CH, t1 - base), next = base + CH;
        if (next < t1) load(stage ^ 1, next, min(CH, t1 - next));
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const float* xs = smem + (size_t)stage * kStage;
        const float *ks = xs + CH * DP, *gs = ks + CH * DP, *vs = gs + CH * DP, *ps = vs + CH * COLS;
        float* dst = out + (size_t)base * H * dv + (size_t)h * dv + j;
        if (WKV) {
            // the read-out is off the state's chain: the sums of four tokens over the lanes run side by side, and a token's
            // rows are read while the one before it is computed
            TokenRows<VPL> row;
            row.template read<SPLIT>(xs, ks, gs, part);
            auto tokens = [&](int first, auto n) {
                constexpr int N = decltype(n)::value;
                float o[N], vv[N], now[N];
#pragma unroll
                for (int u = 0; u < N; ++u) {
                    vv[u] = vs[(first + u) * COLS + cb];
                    now[u] = ps[2 * (first + u)];
                }
#pragma unroll
                for (int u = 0; u < N; ++u) {
                    const TokenRows<VPL> cur = row;
                    const int nt = min(first + u + 1, count - 1);
                    row.template read<SPLIT>(xs + nt * DP, ks + nt * DP, gs + nt * DP, part);
                    float acc[VPL / 4];
#pragma unroll
                    for (int c = 0; c < VPL / 4; ++c) {
                        acc[c] = dot4(S + 4 * c, cur.x[c], 0.f);
                        S[4 * c] = fmaf(cur.g[c].x, S[4 * c], cur.k[c].x * vv[u]);
                        S[4 * c + 1] = fmaf(cur.g[c].y, S[4 * c + 1], cur.k[c].y * vv[u]);
                        S[4 * c + 2] = fmaf(cur.g[c].z, S[4 * c + 2], cur.k[c].z * vv[u]);
                        S[4 * c + 3] = fmaf(cur.g[c].w, S[4 * c + 3], cur.k[c].w * vv[u]);
                    }
                    o[u] = sum_of(acc);
                }
#pragma unroll
                for (int w = SPLIT / 2; w > 0; w >>= 1)
#pragma unroll
                    for (int u = 0; u < N; ++u) o[u] += __shfl_xor_sync(0xffffffffu, o[u], w);
                if (col && part == 0) {
#pragma unroll
                    for (int u = 0; u < N; ++u) dst[(size_t)(first + u) * H * dv] = fmaf(now[u], vv[u], o[u]);
                }
            };
            int tt = 0;
            for (; tt + 4 <= count; tt += 4) tokens(tt, std::integral_constant<int, 4>{});
            for (; tt < count; ++tt) tokens(tt, std::integral_constant<int, 1>{});
        } else {
            TokenRows<VPL> row;
            row.template read<SPLIT>(xs, ks, gs, part);
            for (int tt = 0; tt < count; ++tt) {
                const float2 p = *reinterpret_cast<const float2*>(ps + 2 * tt);      // beta, k.q
                const float vv = vs[tt * COLS + cb];
                float rk[VPL / 4], pq[VPL / 4];
                float4 k4[VPL / 4];
#pragma unroll
                for (int c = 0; c < VPL / 4; ++c) {
                    S[4 * c] *= row.g[c].x;
                    S[4 * c + 1] *= row.g[c].y;
                    S[4 * c + 2] *= row.g[c].z;
                    S[4 * c + 3] *= row.g[c].w;
                    rk[c] = dot4(S + 4 * c, row.k[c], 0.f);
                    pq[c] = dot4(S + 4 * c, row.x[c], 0.f);
                    k4[c] = row.k[c];
                }
                // the next token's rows are on their way while this one's sums run (the last one reads its own again)
                const int nt = min(tt + 1, count - 1);
                row.template read<SPLIT>(xs + nt * DP, ks + nt * DP, gs + nt * DP, part);
                float a = sum_of(rk), b = sum_of(pq);
#pragma unroll
                for (int w = SPLIT / 2; w > 0; w >>= 1) {
                    a += __shfl_xor_sync(0xffffffffu, a, w);
                    b += __shfl_xor_sync(0xffffffffu, b, w);
                }
                const float u = p.x * (vv - a);
#pragma unroll
                for (int c = 0; c < VPL / 4; ++c) {
                    S[4 * c] = fmaf(k4[c].x, u, S[4 * c]);
                    S[4 * c + 1] = fmaf(k4[c].y, u, S[4 * c + 1]);
                    S[4 * c + 2] = fmaf(k4[c].z, u, S[4 * c + 2]);
                    S[4 * c + 3] = fmaf(k4[c].w, u, S[4 * c + 3]);
                }
                if (col && part == 0) dst[(size_t)tt * H * dv] = fmaf(u, p.y, b);
            }
        }
        __syncthreads();                                     // the stage is free before it is filled again
    }
    if (has && col) {
#pragma unroll
        for (int i = 0; i < VPL; ++i) {
            const int row = ((i / 4) * SPLIT + part) * 4 + i % 4;
            if (row < d) st[(size_t)row * dv + j] = S[i];
        }
    }
}

template <int DP, int VPL, bool WKV>
static int launch_channel_scan_vpl(const float* x, const float* k, int xk_stride, const float* g, int g_stride, const float* v,
                                   int v_stride, const float* pairs, int heads_per_key, float* state, const int* query_start_loc,
                                   const int* state_slots, int num_slots, int num_requests, float* out, int H, int d, int dv,
                                   cudaStream_t stream) {
    constexpr int WARPS = channel_warps<VPL>(), COLS = (32 / (DP / VPL)) * WARPS, CH = channel_stage_tokens<DP>();
    constexpr size_t smem = (size_t)2 * (3 * CH * DP + CH * COLS + CH * 2) * sizeof(float);
    static SmemLimit limit;
    if (smem > 48 * 1024)
        if (int rc = raise_smem_limit(limit, channel_scan_kernel<DP, VPL, WKV>, smem, "channel_scan")) return rc;
    auto aligned = [](const float* p, int stride) { return ((uintptr_t)p % 16) == 0 && stride % 4 == 0; };
    const int vec4 = d % 4 == 0 && aligned(x, xk_stride) && aligned(k, xk_stride) && aligned(g, g_stride);
    const int vec4_v = dv % 4 == 0 && aligned(v, v_stride);
    // not as a dependent launch: CTAs that start under the tail of the kernel before them land on the few SMs that have
    // room, several on one, and stay there (a prompt of 2 048 tokens: 0.65 ms instead of 0.38)
    channel_scan_kernel<DP, VPL, WKV><<<dim3(num_requests, H, (dv + COLS - 1) / COLS), WARPS * 32, smem, stream>>>(
        x, k, xk_stride, g, g_stride, v, v_stride, pairs, heads_per_key, vec4, vec4_v, state, query_start_loc, state_slots, num_slots, out,
        H, d, dv);
    return 0;
}

// Values a lane: 8 while the warps that makes are few for the GPU's 592 warp schedulers, then 16, then 32.
template <int DP, bool WKV>
static int launch_channel_scan(const float* x, const float* k, int xk_stride, const float* g, int g_stride, const float* v, int v_stride,
                               const float* pairs, int heads_per_key, float* state, const int* query_start_loc, const int* state_slots,
                               int num_slots, int num_requests, float* out, int H, int d, int dv, cudaStream_t stream) {
    const long long values = (long long)num_requests * H * dv * DP;
#define CIB_CHANNEL(VPL)                                                                                                            \
    return launch_channel_scan_vpl<DP, VPL, WKV>(x, k, xk_stride, g, g_stride, v, v_stride, pairs, heads_per_key, state, query_start_loc, \
                                                 state_slots, num_slots, num_requests, out, H, d, dv, stream)
    if (values <= 8ll * 32 * kChannelFewWarps) CIB_CHANNEL(8);
    if (values <= 16ll * 32 * kChannelManyWarps) CIB_CHANNEL(16);
    CIB_CHANNEL(32);
#undef CIB_CHANNEL
}

// ---- token shift ------------------------------------------------------------------------------------------------------
// out[s, t, :] = h_t + (h_(t-1) - h_t) * mu[s, :] for each of `streams` mixing vectors; the token before a request's first
// row comes from its state (zeros at the start of a sequence).  A block per token; the block of a request's first row,
// the only one that reads the state, leaves the request's last row there.
template <typename T, int V>
__global__ void __launch_bounds__(256)
token_shift_kernel(const T* __restrict__ x, int stride, const float* __restrict__ mu, int streams, float* __restrict__ state,
                   const int* __restrict__ query_start_loc, const int* __restrict__ token_request,
                   const int* __restrict__ state_slots, int num_slots, T* __restrict__ out, int width, int num_tokens) {
    griddep_launch();
    griddep_wait();
    const int t = blockIdx.x;
    const int r = token_request[t];
    const int start = query_start_loc[r], last = query_start_loc[r + 1] - 1;
    const int slot = state_slots[r];
    float* st = slot >= 0 && slot < num_slots ? state + (size_t)slot * width : nullptr;
    const bool first = t == start;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float now[V], before[V], keep[V];
#pragma unroll
        for (int k = 0; k < V; ++k) now[k] = to_f32(x[(size_t)t * stride + i + k]);
#pragma unroll
        for (int k = 0; k < V; ++k) before[k] = !first ? to_f32(x[(size_t)(t - 1) * stride + i + k]) : st ? st[i + k] : 0.f;
        if (first && st) {
#pragma unroll
            for (int k = 0; k < V; ++k) keep[k] = to_f32(x[(size_t)last * stride + i + k]);
#pragma unroll
            for (int k = 0; k < V; ++k) st[i + k] = keep[k];
        }
        for (int s = 0; s < streams; ++s) {
            T* dst = out + ((size_t)s * num_tokens + t) * width + i;
            const float* m = mu + (size_t)s * width + i;
#pragma unroll
            for (int k = 0; k < V; ++k) dst[k] = from_f32<T>(fmaf(before[k] - now[k], m[k], now[k]));
        }
    }
}

}  // namespace cib

using namespace cib;

static dim3 channel_grid(int num_requests, int H, int d, int dv) {
    const int dp = d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : 256;
    const int cols = (32 / (dp / 32)) * kScanWarps;               // columns of the matrix a block holds
    return dim3(num_requests, H, (dv + cols - 1) / cols);
}

// qkv: float32 rows [q (G d) | k (G d) | v (H dv)]; zb: beta logits [tokens][H]; za: decay logits [tokens][H d]; a_log [H],
// dt_bias [H d]; state [slots][H][d * dv]; out float32 [tokens][H dv].  decay (float32 [tokens][H d], 16-byte aligned) and pairs
// (float32 [tokens][H][2]): room for the two-launch form, or null for the one-launch form (steps of single tokens).
extern "C" int cib_channel_delta_scan(const float* qkv, int qkv_stride, int G, const float* zb, int zb_stride, const float* za,
                                      int za_stride, const void* a_log, const void* dt_bias, int vec_dtype, float* state,
                                      const int* query_start_loc, const int* state_slots, int num_slots, int num_requests,
                                      int num_tokens, float* decay, float* pairs, float* out, int H, int d, int dv,
                                      cudaStream_t stream) {
    CIB_REQUIRE(G > 0 && H > 0 && H % G == 0 && d > 0 && dv > 0, "channel_delta_scan: bad sizes");
    CIB_REQUIRE(d <= 256, "channel_delta_scan: key size %d is beyond 256", d);
    if (num_requests == 0 || num_tokens == 0) return 0;
    AnyVec al{a_log, vec_dtype == kBF16}, db{dt_bias, vec_dtype == kBF16};
    const dim3 grid = channel_grid(num_requests, H, d, dv);
    CIB_REQUIRE((decay == nullptr) == (pairs == nullptr), "channel_delta_scan: the two-launch form needs both rooms");
    if (decay) {
        const long long total = (long long)num_tokens * H;
        launch_pdl(channel_delta_gates_kernel, dim3((unsigned)((total + kGatherWarps - 1) / kGatherWarps)), dim3(kGatherWarps * 32), 0, stream,
                   prompt_pdl(), qkv, qkv_stride, G, zb, zb_stride, za, za_stride, al, db, decay, pairs, H, d, total);
        CIB_LAUNCH_CHECK("channel_delta_gates");
        int rc = 0;
        CIB_SCAN_DISPATCH(d, (rc = launch_channel_scan<DP, false>(qkv, qkv + (size_t)G * d, qkv_stride, decay, H * d, qkv + (size_t)2 * G * d, qkv_stride, pairs, H / G, state, query_start_loc, state_slots, num_slots, num_requests, out, H, d, dv, stream)));
        if (rc) return rc;
        CIB_LAUNCH_CHECK("channel_delta_scan");
        return 0;
    }
    CIB_SCAN_DISPATCH(d, (launch_pdl(channel_delta_scan_kernel<DP>, grid, dim3(kScanWarps * 32), 0, stream, prompt_pdl(), qkv, qkv_stride, G, zb, zb_stride, za, za_stride, al, db, state, query_start_loc, state_slots, num_slots, out, H, d, dv)));
    CIB_LAUNCH_CHECK("channel_delta_scan");
    return 0;
}

// r, k [tokens][H d], v [tokens][H dv]: rows `stride` apart, of one type; zw: decay logits float32 [tokens][H d]; w0, bonus
// [H d]; state [slots][H][d * dv]; out float32 [tokens][H dv].  rows (float32 [tokens][H (3 d + dv)], 16-byte aligned) and pairs
// (float32 [tokens][H][2]): room for the two-launch form, or null for the one-launch form (steps of single tokens).
extern "C" int cib_wkv_scan(const void* r, const void* k, const void* v, int dtype, int stride, const float* zw, int zw_stride,
                            const void* w0, const void* bonus, int vec_dtype, float* state, const int* query_start_loc,
                            const int* state_slots, int num_slots, int num_requests, int num_tokens, float* rows, float* pairs,
                            float* out, int H, int d, int dv, cudaStream_t stream) {
    CIB_REQUIRE(H > 0 && d > 0 && dv > 0, "wkv_scan: bad sizes");
    CIB_REQUIRE((rows == nullptr) == (pairs == nullptr), "wkv_scan: the two-launch form needs both rooms");
    CIB_REQUIRE(d <= 256, "wkv_scan: key size %d is beyond 256", d);
    if (num_requests == 0 || num_tokens == 0) return 0;
    AnyVec w{w0, vec_dtype == kBF16}, b{bonus, vec_dtype == kBF16};
    const dim3 grid = channel_grid(num_requests, H, d, dv);
    if (rows) {
        const long long total = (long long)num_tokens * H;
        const dim3 blocks((unsigned)((total + kGatherWarps - 1) / kGatherWarps));
        if (dtype == kF32) launch_pdl(wkv_rows_kernel<float>, blocks, dim3(kGatherWarps * 32), 0, stream, prompt_pdl(), (const float*)r, (const float*)k, (const float*)v, stride, zw, zw_stride, w, b, rows, pairs, H, d, dv, total);
        else if (dtype == kBF16) launch_pdl(wkv_rows_kernel<__nv_bfloat16>, blocks, dim3(kGatherWarps * 32), 0, stream, prompt_pdl(), (const __nv_bfloat16*)r, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, stride, zw, zw_stride, w, b, rows, pairs, H, d, dv, total);
        else CIB_REQUIRE(false, "wkv_scan: bad dtype %d", dtype);
        CIB_LAUNCH_CHECK("wkv_rows");
        const int width = H * (3 * d + dv);
        int rc = 0;
        CIB_SCAN_DISPATCH(d, (rc = launch_channel_scan<DP, true>(rows, rows + (size_t)H * d, width, rows + (size_t)2 * H * d, width, rows + (size_t)3 * H * d, width, pairs, 1, state, query_start_loc, state_slots, num_slots, num_requests, out, H, d, dv, stream)));
        if (rc) return rc;
        CIB_LAUNCH_CHECK("wkv_scan");
        return 0;
    }
    if (dtype == kF32) {
        CIB_SCAN_DISPATCH(d, (launch_pdl(wkv_scan_kernel<float, DP>, grid, dim3(kScanWarps * 32), 0, stream, prompt_pdl(), (const float*)r, (const float*)k, (const float*)v, stride, zw, zw_stride, w, b, state, query_start_loc, state_slots, num_slots, out, H, d, dv)));
    } else if (dtype == kBF16) {
        CIB_SCAN_DISPATCH(d, (launch_pdl(wkv_scan_kernel<__nv_bfloat16, DP>, grid, dim3(kScanWarps * 32), 0, stream, prompt_pdl(), (const __nv_bfloat16*)r, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, stride, zw, zw_stride, w, b, state, query_start_loc, state_slots, num_slots, out, H, d, dv)));
    } else {
        CIB_REQUIRE(false, "wkv_scan: bad dtype %d", dtype);
    }
    CIB_LAUNCH_CHECK("wkv_scan");
    return 0;
}

// x: [tokens][width] rows; mu float32 [streams][width]; state float32 [slots][width]; out [streams][tokens][width].
extern "C" int cib_token_shift(const void* x, int dtype, int stride, const float* mu, int streams, float* state,
                               const int* query_start_loc, const int* token_request, const int* state_slots, int num_slots,
                               void* out, int width, int num_tokens, cudaStream_t stream) {
    CIB_REQUIRE(streams > 0 && width > 0 && stride >= width && num_tokens >= 0, "token_shift: bad sizes");
    if (num_tokens == 0) return 0;
    const bool pdl = prompt_pdl();
#define CIB_SHIFT(T, V)                                                                                                        \
    launch_pdl(token_shift_kernel<T, V>, dim3(num_tokens), dim3(256), 0, stream, pdl, (const T*)x, stride, mu, streams, state,   \
               query_start_loc, token_request, state_slots, num_slots, (T*)out, width, num_tokens)
    if (dtype == kF32) CIB_SHIFT(float, 1);
    else if (dtype == kBF16 && width % 2 == 0 && stride % 2 == 0) CIB_SHIFT(__nv_bfloat16, 2);
    else if (dtype == kBF16) CIB_SHIFT(__nv_bfloat16, 1);
    else CIB_REQUIRE(false, "token_shift: bad dtype %d", dtype);
#undef CIB_SHIFT
    CIB_LAUNCH_CHECK("token_shift");
    return 0;
}
