// Recurrences whose decay is a vector: every key channel (row of a head's matrix) fades at a rate of its own per token.
// The gated delta rule in that form, and the time mixing of the RWKV family with its token shift and its bonus for the
// current token.  Layout of requests, slots and columns as in recurrent.cu; everything here is 32-bit.
//
// Per head, decay g (one number per row of S):
//   delta: S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   wkv:   o = (S + diag(b) k v^T)^T r;  S <- diag(g) S + k v^T          (b: the bonus, a number per head and channel)
// Column j of S depends on nothing but itself, the token's rows and v_j.
#include "mma_utils.cuh"
#include "scan_utils.cuh"

namespace cib {

template <int DP> constexpr int channel_chunk() { return DP > 128 ? 8 : 16; }        // tokens staged at a time (48 KB)

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
            const float* kseg = &ksm[tt][part * 36];
            const float* qseg = &qsm[tt][part * 36];
            const float* gseg = &gsm[tt][part * 36];
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
            const float u = bsm[tt] * (vsm[tt][cb] - rk);
#pragma unroll
            for (int i = 0; i < 32; i += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(kseg + i);
                S[i] = fmaf(k4.x, u, S[i]);
                S[i + 1] = fmaf(k4.y, u, S[i + 1]);
                S[i + 2] = fmaf(k4.z, u, S[i + 2]);
                S[i + 3] = fmaf(k4.w, u, S[i + 3]);
            }
            if (col && part == 0) out[(size_t)(base + tt) * H * dv + (size_t)h * dv + j] = pq + u * kq;
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
            const float* kseg = &ksm[tt][part * 36];
            const float* rseg = &rsm[tt][part * 36];
            const float* gseg = &gsm[tt][part * 36];
            const float v = vsm[tt][cb];
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
            const float o = split_sum<SPLIT>((o4[0] + o4[1]) + (o4[2] + o4[3]));
            if (col && part == 0) out[(size_t)(base + tt) * H * dv + (size_t)h * dv + j] = fmaf(now, v, o);
        }
    }
    if (has && col) {
#pragma unroll
        for (int i = 0; i < 32; ++i)
            if (i0 + i < d) st[(size_t)(i0 + i) * dv + j] = S[i];
    }
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
// dt_bias [H d]; state [slots][H][d * dv]; out float32 [tokens][H dv].
extern "C" int cib_channel_delta_scan(const float* qkv, int qkv_stride, int G, const float* zb, int zb_stride, const float* za,
                                      int za_stride, const void* a_log, const void* dt_bias, int vec_dtype, float* state,
                                      const int* query_start_loc, const int* state_slots, int num_slots, int num_requests,
                                      int num_tokens, float* out, int H, int d, int dv, cudaStream_t stream) {
    CIB_REQUIRE(G > 0 && H > 0 && H % G == 0 && d > 0 && dv > 0, "channel_delta_scan: bad sizes");
    CIB_REQUIRE(d <= 256, "channel_delta_scan: key size %d is beyond 256", d);
    if (num_requests == 0 || num_tokens == 0) return 0;
    AnyVec al{a_log, vec_dtype == kBF16}, db{dt_bias, vec_dtype == kBF16};
    const dim3 grid = channel_grid(num_requests, H, d, dv);
    CIB_SCAN_DISPATCH(d, (launch_pdl(channel_delta_scan_kernel<DP>, grid, dim3(kScanWarps * 32), 0, stream, prompt_pdl(), qkv, qkv_stride, G, zb, zb_stride, za, za_stride, al, db, state, query_start_loc, state_slots, num_slots, out, H, d, dv)));
    CIB_LAUNCH_CHECK("channel_delta_scan");
    return 0;
}

// r, k [tokens][H d], v [tokens][H dv]: rows `stride` apart, of one type; zw: decay logits float32 [tokens][H d]; w0, bonus
// [H d]; state [slots][H][d * dv]; out float32 [tokens][H dv].
extern "C" int cib_wkv_scan(const void* r, const void* k, const void* v, int dtype, int stride, const float* zw, int zw_stride,
                            const void* w0, const void* bonus, int vec_dtype, float* state, const int* query_start_loc,
                            const int* state_slots, int num_slots, int num_requests, int num_tokens, float* out, int H, int d,
                            int dv, cudaStream_t stream) {
    CIB_REQUIRE(H > 0 && d > 0 && dv > 0, "wkv_scan: bad sizes");
    CIB_REQUIRE(d <= 256, "wkv_scan: key size %d is beyond 256", d);
    if (num_requests == 0 || num_tokens == 0) return 0;
    AnyVec w{w0, vec_dtype == kBF16}, b{bonus, vec_dtype == kBF16};
    const dim3 grid = channel_grid(num_requests, H, d, dv);
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
