// A short causal convolution over time per channel, for mixers whose rows pass one before their recurrence.
//
//   u_t = x_t + in_bias;   y_t = act(bias + sum_j taps[K - 1 - j] * u_(t - j)),   act the identity or SiLU
//
// Requests, slots and the order of tokens as in recurrent.cu.  Inputs before a step's rows come from the request's state
// ([K - 1][C], oldest first, input bias included); before the start of a sequence they are zero (the state of a new
// request is).  A thread walks a few consecutive tokens of V neighbouring channels with the last inputs in registers,
// so that a row is read once (a step of few tokens gives every token a thread of its own); at a request's first row the registers are filled from its state.  With
// `one_token_each` the thread that reads a request's state also moves it on; otherwise `conv_state_update_kernel`
// (recurrent.cu) does that after this launch.  Sums and activation 32-bit, one rounding at the end.
#include <algorithm>

#include "mma_utils.cuh"

namespace cib {

constexpr int kConvTokens = 8;           // tokens a thread walks (one in a step of few tokens)
constexpr int kConvFewTokens = 256;
constexpr int kConvMaxTaps = 16;

template <typename T, int V> __device__ __forceinline__ void load_row(const T* p, float (&v)[V]) {
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] = to_f32(p[k]);
}
template <> __device__ __forceinline__ void load_row<float, 4>(const float* p, float (&v)[4]) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
}
template <> __device__ __forceinline__ void load_row<__nv_bfloat16, 4>(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&t.x), b = *reinterpret_cast<const __nv_bfloat162*>(&t.y);
    v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
}
template <typename T, int V> __device__ __forceinline__ void store_row(T* p, const float (&v)[V]) {
#pragma unroll
    for (int k = 0; k < V; ++k) p[k] = from_f32<T>(v[k]);
}
template <> __device__ __forceinline__ void store_row<float, 4>(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void store_row<__nv_bfloat16, 4>(__nv_bfloat16* p, const float (&v)[4]) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
}

// KT: taps held in registers, K <= KT (a tap beyond K is zero); TB: tokens a thread walks.
template <typename TI, typename TO, int V, int KT, int TB>
__global__ void __launch_bounds__(128)
short_conv_kernel(const TI* __restrict__ x, int stride, const float* __restrict__ taps, int K, const float* __restrict__ in_bias,
                  const float* __restrict__ bias, int silu, float* __restrict__ state, const int* __restrict__ query_start_loc,
                  const int* __restrict__ token_request, const int* __restrict__ state_slots, int num_slots, TO* __restrict__ out,
                  int out_stride, int C, int num_tokens, int one_token_each) {
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    griddep_launch();
    if (c >= C) return;
    float w[KT][V], ib[V], ob[V];                     // weights: not written by the kernel before this one
#pragma unroll
    for (int j = 0; j < KT; ++j)
#pragma unroll
        for (int k = 0; k < V; ++k) w[j][k] = j < K ? taps[(size_t)(K - 1 - j) * C + c + k] : 0.f;
#pragma unroll
    for (int k = 0; k < V; ++k) {
        ib[k] = in_bias ? in_bias[c + k] : 0.f;
        ob[k] = bias ? bias[c + k] : 0.f;
    }
    griddep_wait();
    const int t0 = blockIdx.x * TB, t1 = min(num_tokens, t0 + TB);
    if constexpr (TB > 1) {
        // all of the tokens and what precedes them in one request: every row is asked for before the first is used
        const int r = token_request[t0];
        if (t1 == t0 + TB && t0 - (KT - 1) >= query_start_loc[r] && t1 <= query_start_loc[r + 1]) {
            float u[TB + KT - 1][V];
#pragma unroll
            for (int i = 0; i < TB + KT - 1; ++i) load_row<TI, V>(x + (size_t)(t0 - (KT - 1) + i) * stride + c, u[i]);
#pragma unroll
            for (int i = 0; i < TB + KT - 1; ++i)
#pragma unroll
                for (int k = 0; k < V; ++k) u[i][k] += ib[k];
#pragma unroll
            for (int i = 0; i < TB; ++i) {
                float y[V];
#pragma unroll
                for (int k = 0; k < V; ++k) {
                    float s = 0.f;
#pragma unroll
                    for (int j = 0; j < KT; ++j) s = fmaf(w[j][k], u[i + KT - 1 - j][k], s);
                    s += ob[k];
                    y[k] = silu ? s / (1.f + expf(-s)) : s;
                }
                store_row<TO, V>(out + (size_t)(t0 + i) * out_stride + c, y);
            }
            return;
        }
    }
    float win[KT][V];                                 // win[j]: the input j tokens back
    for (int t = t0; t < t1; ++t) {
        const int r = token_request[t];
        const int start = query_start_loc[r];
        const int slot = state_slots[r];
        float* st = (K > 1 && slot >= 0 && slot < num_slots) ? state + (size_t)slot * (K - 1) * C + c : nullptr;
        if (t == t0 || t == start) {
#pragma unroll
            for (int j = KT - 1; j >= 1; --j) {
                const int tt = t - j;
#pragma unroll
                for (int k = 0; k < V; ++k) win[j - 1][k] = 0.f;      // shifted to place j below
                if (j >= K) continue;
                if (tt >= start) {
                    load_row<TI, V>(x + (size_t)tt * stride + c, win[j - 1]);
#pragma unroll
                    for (int k = 0; k < V; ++k) win[j - 1][k] += ib[k];
                } else if (st) {
                    load_row<float, V>(st + (size_t)(K - 1 - (start - tt)) * C, win[j - 1]);
                }
            }
        }
#pragma unroll
        for (int j = KT - 1; j >= 1; --j)
#pragma unroll
            for (int k = 0; k < V; ++k) win[j][k] = win[j - 1][k];
        load_row<TI, V>(x + (size_t)t * stride + c, win[0]);
        float y[V];
#pragma unroll
        for (int k = 0; k < V; ++k) {
            win[0][k] += ib[k];
            float s = 0.f;
#pragma unroll
            for (int j = 0; j < KT; ++j) s = fmaf(w[j][k], win[j][k], s);
            s += ob[k];
            y[k] = silu ? s / (1.f + expf(-s)) : s;
        }
        store_row<TO, V>(out + (size_t)t * out_stride + c, y);
        if (one_token_each && st) {                   // this thread alone reads and writes these channels of the slot
#pragma unroll
            for (int j = 0; j < KT; ++j)
                if (j < K - 1) store_row<float, V>(st + (size_t)(K - 2 - j) * C, win[j]);
        }
    }
}

}  // namespace cib

using namespace cib;

// x [tokens][>= C] rows `stride` apart; taps float32 [K][C] (the last row is the current token's); in_bias, bias float32 [C] or
// null; state float32 [slots][max(K - 1, 1)][C]; out [tokens][>= C] rows `out_stride` apart.
extern "C" int cib_short_conv(const void* x, int dtype, int stride, const float* taps, int K, const float* in_bias, const float* bias,
                              int silu, float* state, const int* query_start_loc, const int* token_request, const int* state_slots,
                              int num_slots, void* out, int out_dtype, int out_stride, int C, int num_tokens, int one_token_each,
                              cudaStream_t stream) {
    CIB_REQUIRE(C > 0 && K >= 1 && stride >= C && out_stride >= C && num_tokens >= 0, "short_conv: bad sizes");
    CIB_REQUIRE(K <= kConvMaxTaps, "short_conv: %d taps are beyond %d", K, kConvMaxTaps);
    CIB_REQUIRE(K == 1 || state, "short_conv: the state is missing");
    if (num_tokens == 0) return 0;
    const size_t in_bytes = (dtype == kF32 ? 16 : 8), out_bytes = (out_dtype == kF32 ? 16 : 8);
    const bool v4 = C % 4 == 0 && stride % 4 == 0 && out_stride % 4 == 0 && (uintptr_t)x % in_bytes == 0 && (uintptr_t)out % out_bytes == 0 &&
                    (uintptr_t)state % 16 == 0;
    const int per = v4 ? 4 : 1;
    const int walk = num_tokens <= kConvFewTokens || K > 4 ? 1 : kConvTokens;
    const dim3 grid((unsigned)((num_tokens + walk - 1) / walk), (unsigned)((C / per + 127) / 128));
    CIB_REQUIRE(grid.y <= 65535, "short_conv: %d channels are beyond this kernel", C);
    const bool pdl = prompt_pdl();
    cudaError_t e = cudaErrorInvalidValue;
#define CIB_CONV(TI, TO, V, KT, TB)                                                                                                   \
    e = launch_pdl(short_conv_kernel<TI, TO, V, KT, TB>, grid, dim3(128), 0, stream, pdl, (const TI*)x, stride, taps, K, in_bias, bias, silu,  \
                   state, query_start_loc, token_request, state_slots, num_slots, (TO*)out, out_stride, C, num_tokens, one_token_each)
#define CIB_CONV_K(TI, TO, V)                       \
    do {                                            \
        if (walk > 1) CIB_CONV(TI, TO, V, 4, kConvTokens);      \
        else if (K <= 4) CIB_CONV(TI, TO, V, 4, 1);             \
        else CIB_CONV(TI, TO, V, kConvMaxTaps, 1);              \
    } while (0)
#define CIB_CONV_V(TI, TO)                          \
    do {                                            \
        if (v4) CIB_CONV_K(TI, TO, 4);              \
        else CIB_CONV_K(TI, TO, 1);                 \
    } while (0)
    if (dtype == kF32 && out_dtype == kF32) CIB_CONV_V(float, float);
    else if (dtype == kF32 && out_dtype == kBF16) CIB_CONV_V(float, __nv_bfloat16);
    else if (dtype == kBF16 && out_dtype == kBF16) CIB_CONV_V(__nv_bfloat16, __nv_bfloat16);
    else CIB_REQUIRE(false, "short_conv: bad dtypes %d -> %d", dtype, out_dtype);
#undef CIB_CONV_V
#undef CIB_CONV_K
#undef CIB_CONV
    if (e != cudaSuccess) {
        set_error("short_conv: launch failed: %s", cudaGetErrorString(e));
        return -2;
    }
    return 0;
}
