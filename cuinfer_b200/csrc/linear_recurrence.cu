// A gated linear recurrence with one number of state per channel (the RG-LRU of Griffin).
//
// For the convolved rows u of C channels in `blocks` equal parts of b, with a pair of square matrices per part:
//
//   r = sigmoid(Ra u + ra);  i = sigmoid(Ri u + ri);  log a = -8 r softplus(lam)
//   S <- a S + sqrt(1 - a^2) i u;    out = out_scale * S * gelu_tanh(y + y_bias)
//
// Requests, slots and the order of tokens as in recurrent.cu.  Gates, decay, state and what follows are 32-bit;
// a slow decay is kept as a - 1, so that what it takes off, and sqrt(1 - a^2), keep their digits over thousands of tokens.
//
//  * lru_gates_mma (bfloat16 rows, blocks in multiples of 32): both gate products of 64 tokens x 64 channels on the tensor
//    cores over one tile of u, decay and input as the epilogue: pairs (decay, sqrt(1 - a^2) i u) per token and channel.
//  * lru_gates: the same pairs from logits another product left (32-bit, any sizes).
//  * lru_scan: the recurrence over the pairs.  S_t is a composition of maps S -> a S + c, which is associative: the warps of a
//    block take consecutive parts of a request's tokens for 32 channels (a lane a channel), each composes its part's map,
//    and after one exchange walks it from its own starting state.
//  * lru_decode (steps of single tokens): gate products, decay, update and output in one launch; a warp reads a channel's
//    two matrix rows once for eight tokens.
#include "mma_utils.cuh"
#include "scan_utils.cuh"

namespace cib {

__device__ __forceinline__ float gelu_tanhf_(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// Decay and what joins the state, from the gates' logits.  The decay a is encoded by its sign: x <= 0 means a = 1 + x (slow),
// x > 0 means a = x.
constexpr float kSlowLog = -0.5f;
__device__ __forceinline__ float2 lru_pair(float zr, float zi, float u, float sp) {
    const float log_a = -8.f * sigmoidf_(zr) * sp;
    float x, rest;                                       // rest: 1 - a^2
    if (log_a >= kSlowLog) {
        x = expm1f(log_a);
        rest = -x * (2.f + x);
    } else {
        x = fmaxf(expf(log_a), 1e-37f);
        rest = (1.f - x) * (1.f + x);
    }
    return make_float2(x, sqrtf(rest) * sigmoidf_(zi) * u);
}
__device__ __forceinline__ float lru_apply(float x, float S, float c) { return fmaf(x <= 0.f ? 1.f : 0.f, S, fmaf(x, S, c)); }

constexpr int kLM = 64, kLN = 64, kLK = 32, kLStages = 3, kLLd = kLK + 8;

// w [blocks][2 b][b]: a part's rows of Ra, then of Ri.  grid (token tiles, blocks * channel tiles).
__global__ void __launch_bounds__(128)
lru_gates_mma_kernel(const __nv_bfloat16* __restrict__ u, int u_stride, const __nv_bfloat16* __restrict__ w, const float* __restrict__ bias,
                     const float* __restrict__ sp, float2* __restrict__ pairs, int C, int b, int num_tokens) {
    __shared__ __align__(16) __nv_bfloat16 sA[kLStages][kLM][kLLd];
    __shared__ __align__(16) __nv_bfloat16 sB[kLStages][2][kLN][kLLd];
    __shared__ __align__(8) float s_bias[2][kLN], s_sp[kLN];       // of this tile's channels
    griddep_launch();
    griddep_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int tiles = (b + kLN - 1) / kLN;
    const int block = blockIdx.y / tiles, n0 = (blockIdx.y % tiles) * kLN, m0 = blockIdx.x * kLM;
    const int rows = min(kLM, num_tokens - m0);
    if (tid < kLN) {
        const int c = block * b + min(n0 + tid, b - 1);
        s_bias[0][tid] = bias[c];
        s_bias[1][tid] = bias[C + c];
        s_sp[tid] = sp[c];
    }
    const __nv_bfloat16* wb = w + (size_t)block * 2 * b * b;
    const __nv_bfloat16* a = u + (size_t)m0 * u_stride + (size_t)block * b;
    auto load = [&](int stage, int k0) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            const int idx = tid + c * 128, row = idx >> 2, k = k0 + (idx & 3) * 8;
            const bool ok = row < rows;
            cp_async16(&sA[stage][row][(idx & 3) * 8], a + (ok ? (size_t)row * u_stride + k : 0), ok);
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int idx = tid + c * 128, half = idx >> 8, row = (idx >> 2) & 63, k = k0 + (idx & 3) * 8;
            const bool ok = n0 + row < b;
            cp_async16(&sB[stage][half][row][(idx & 3) * 8], wb + (ok ? (size_t)(half * b + n0 + row) * b + k : 0), ok);
        }
    };
    float acc[2][kLN / 8][4];
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int i = 0; i < kLN / 8; ++i) acc[h][i][0] = acc[h][i][1] = acc[h][i][2] = acc[h][i][3] = 0.f;
    const int steps = b / kLK;
#pragma unroll
    for (int s = 0; s < kLStages - 1; ++s) {
        if (s < steps) load(s, s * kLK);
        cp_async_commit();
    }
    const int mat = lane >> 3, rr = lane & 7;
    for (int ks = 0; ks < steps; ++ks) {
        cp_async_wait<kLStages - 2>();
        __syncthreads();
        if (ks + kLStages - 1 < steps) load((ks + kLStages - 1) % kLStages, (ks + kLStages - 1) * kLK);
        cp_async_commit();
        const int st = ks % kLStages;
#pragma unroll
        for (int kk = 0; kk < kLK / 16; ++kk) {
            uint32_t af[4];
            ldmatrix_x4(af, smem_u32(&sA[st][warp * 16 + (mat & 1) * 8 + rr][kk * 16 + (mat >> 1) * 8]));
#pragma unroll
            for (int h = 0; h < 2; ++h)
#pragma unroll
                for (int np = 0; np < kLN / 16; ++np) {
                    uint32_t bf[4];
                    ldmatrix_x4(bf, smem_u32(&sB[st][h][np * 16 + (mat >> 1) * 8 + rr][kk * 16 + (mat & 1) * 8]));
                    mma_bf16_16816(acc[h][2 * np], af, bf[0], bf[1]);
                    mma_bf16_16816(acc[h][2 * np + 1], af, bf[2], bf[3]);
                }
        }
    }
    cp_async_wait<0>();
    const int qrow = lane >> 2, quad = lane & 3;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int row = warp * 16 + qrow + 8 * half;
        if (row >= rows) continue;
        const size_t t = (size_t)(m0 + row);
        const __nv_bfloat16* ur = u + t * u_stride + (size_t)block * b + n0;
        float4* dst = reinterpret_cast<float4*>(pairs + t * C + (size_t)block * b + n0);
        __nv_bfloat162 uv[kLN / 8];                      // all of the row's inputs are on their way before the first is used
#pragma unroll
        for (int j = 0; j < kLN / 8; ++j)
            if (n0 + j * 8 < b) uv[j] = *reinterpret_cast<const __nv_bfloat162*>(ur + j * 8 + quad * 2);
#pragma unroll
        for (int j = 0; j < kLN / 8; ++j) {
            const int col = j * 8 + quad * 2;            // b is a multiple of 32: a pair of columns is inside or outside
            if (n0 + col >= b) continue;
            const float2 br = *reinterpret_cast<const float2*>(&s_bias[0][col]), bi = *reinterpret_cast<const float2*>(&s_bias[1][col]);
            const float2 rate = *reinterpret_cast<const float2*>(&s_sp[col]);
            const float2 p = lru_pair(acc[0][j][2 * half] + br.x, acc[1][j][2 * half] + bi.x, __low2float(uv[j]), rate.x);
            const float2 q = lru_pair(acc[0][j][2 * half + 1] + br.y, acc[1][j][2 * half + 1] + bi.y, __high2float(uv[j]), rate.y);
            dst[col / 2] = make_float4(p.x, p.y, q.x, q.y);
        }
    }
}

// logits float32 [tokens][blocks][2 b]: a part's values of Ra u, then of Ri u.
template <typename T>
__global__ void lru_gates_kernel(const T* __restrict__ u, int u_stride, const float* __restrict__ logits, const float* __restrict__ bias,
                                 const float* __restrict__ sp, float2* __restrict__ pairs, int C, int b, long long total) {
    const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= total) return;
    const long long t = e / C;
    const int c = (int)(e - t * C), block = c / b, col = c - block * b;
    const float* z = logits + t * 2 * C + (size_t)block * 2 * b;
    pairs[e] = lru_pair(z[col] + bias[c], z[b + col] + bias[C + c], to_f32(u[t * u_stride + c]), sp[c]);
}

constexpr int kLruMaxWarps = 32;
constexpr int kLruUnroll = 8;

template <typename T>
__global__ void __launch_bounds__(kLruMaxWarps * 32)
lru_scan_kernel(const float2* __restrict__ pairs, const T* __restrict__ y, int y_stride, const float* __restrict__ y_bias, float out_scale,
                float* __restrict__ state, const int* __restrict__ query_start_loc, const int* __restrict__ state_slots, int num_slots,
                T* __restrict__ out, int C) {
    __shared__ float sa[kLruMaxWarps][32], sc[kLruMaxWarps][32];
    const int lane = threadIdx.x, warp = threadIdx.y, warps = blockDim.y;
    const int r = blockIdx.y, c = blockIdx.x * 32 + lane;
    griddep_launch();
    griddep_wait();
    const int t0 = query_start_loc[r], t1 = query_start_loc[r + 1];
    if (t1 <= t0) return;
    const bool live = c < C;
    const int slot = state_slots[r];
    float* st = slot >= 0 && slot < num_slots && live ? state + (size_t)slot * C + c : nullptr;
    float S = st ? *st : 0.f;
    const int per = (t1 - t0 + warps - 1) / warps;
    const int begin = min(t1, t0 + warp * per), end = min(t1, begin + per);
    const float2* src = pairs + (live ? c : 0);
    float a = 1.f, add = 0.f;
    for (int t = begin; t < end; t += kLruUnroll) {
        float2 p[kLruUnroll];
#pragma unroll
        for (int k = 0; k < kLruUnroll; ++k) p[k] = t + k < end ? src[(size_t)(t + k) * C] : make_float2(0.f, 0.f);
#pragma unroll
        for (int k = 0; k < kLruUnroll; ++k) {
            a = lru_apply(p[k].x, a, 0.f);
            add = lru_apply(p[k].x, add, p[k].y);
        }
    }
    sa[warp][lane] = a;
    sc[warp][lane] = add;
    __syncthreads();
    if (begin >= end || !live) return;
    for (int w = 0; w < warp; ++w) S = fmaf(sa[w][lane], S, sc[w][lane]);
    const float bias = y_bias[c];
    for (int t = begin; t < end; t += kLruUnroll) {
        float2 p[kLruUnroll];
        float g[kLruUnroll];
#pragma unroll
        for (int k = 0; k < kLruUnroll; ++k) {
            p[k] = t + k < end ? src[(size_t)(t + k) * C] : make_float2(0.f, 0.f);
            g[k] = t + k < end ? to_f32(y[(size_t)(t + k) * y_stride + c]) : 0.f;
        }
#pragma unroll
        for (int k = 0; k < kLruUnroll; ++k) {
            if (t + k >= end) break;
            S = lru_apply(p[k].x, S, p[k].y);
            out[(size_t)(t + k) * C + c] = from_f32<T>(out_scale * S * gelu_tanhf_(g[k] + bias));
        }
    }
    if (end == t1 && st) *st = S;                        // every warp has read the state before the exchange
}

constexpr int kLruTokens = 8, kLruDecodeWarps = 8;

// One token per request (token t is request t's).  grid (blocks, channel tiles of a block): a warp a channel.  The sixteen sums
// of a channel over eight tokens are reduced by halves: at every step a lane gives one half of its sums away and adds to
// the other, so that lane l ends with sum l / 2.
template <typename T, bool VEC>
__global__ void __launch_bounds__(kLruDecodeWarps * 32)
lru_decode_kernel(const T* __restrict__ u, int u_stride, const T* __restrict__ w, const float* __restrict__ bias, const float* __restrict__ sp,
                  const T* __restrict__ y, int y_stride, const float* __restrict__ y_bias, float out_scale, float* __restrict__ state,
                  const int* __restrict__ state_slots, int num_slots, T* __restrict__ out, int C, int b, int num_tokens) {
    extern __shared__ __align__(16) float us[];          // [kLruTokens][b]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int block = blockIdx.x;
    const int col = blockIdx.y * kLruDecodeWarps + warp, c = block * b + min(col, b - 1);
    const T* wr = w + (size_t)block * 2 * b * b + (size_t)min(col, b - 1) * b;
    const T* wi = wr + (size_t)b * b;
    griddep_launch();
    // weights: not written by the kernel before this one
    constexpr int AHEAD = 4;
    uint32_t first_r[AHEAD], first_i[AHEAD];
    if constexpr (VEC) {
#pragma unroll
        for (int q = 0; q < AHEAD; ++q) {
            const int k = q * 64 + lane * 2;
            first_r[q] = k < b ? *reinterpret_cast<const uint32_t*>(wr + k) : 0u;
            first_i[q] = k < b ? *reinterpret_cast<const uint32_t*>(wi + k) : 0u;
        }
    }
    const float br = bias[c], bi = bias[C + c], rate = sp[c], yb = y_bias[c];
    griddep_wait();
    for (int tb = 0; tb < num_tokens; tb += kLruTokens) {
        const int count = min(kLruTokens, num_tokens - tb);
        // lane 4 tt takes token tt: what it needs is on its way before the products
        const int mine = tb + (lane >> 2);
        const bool finish = (lane & 3) == 0 && mine < num_tokens && col < b;
        float* st = nullptr;
        float before = 0.f, gate = 0.f;
        if (finish) {
            const int slot = state_slots[mine];
            st = slot >= 0 && slot < num_slots ? state + (size_t)slot * C + c : nullptr;
            before = st ? *st : 0.f;
            gate = to_f32(y[(size_t)mine * y_stride + c]);
        }
        __syncthreads();
        for (int k = threadIdx.x; k < b; k += blockDim.x) {
            const T* src = u + (size_t)tb * u_stride + (size_t)block * b + k;
            float x[kLruTokens];
#pragma unroll
            for (int tt = 0; tt < kLruTokens; ++tt) x[tt] = tt < count ? to_f32(src[(size_t)tt * u_stride]) : 0.f;
#pragma unroll
            for (int tt = 0; tt < kLruTokens; ++tt) us[tt * b + k] = x[tt];
        }
        __syncthreads();
        float v[2 * kLruTokens];                         // [token][Ra, Ri]
#pragma unroll
        for (int i = 0; i < 2 * kLruTokens; ++i) v[i] = 0.f;
        if constexpr (VEC) {                             // bfloat16, b even: two neighbouring values a lane and load
            auto pair = [&](int k, uint32_t vr, uint32_t vi) {
                const float2 fr = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&vr));
                const float2 fi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&vi));
#pragma unroll
                for (int tt = 0; tt < kLruTokens; ++tt) {
                    const float2 x = *reinterpret_cast<const float2*>(us + tt * b + k);
                    v[2 * tt] = fmaf(fr.x, x.x, fmaf(fr.y, x.y, v[2 * tt]));
                    v[2 * tt + 1] = fmaf(fi.x, x.x, fmaf(fi.y, x.y, v[2 * tt + 1]));
                }
            };
#pragma unroll
            for (int q = 0; q < AHEAD; ++q)
                if (q * 64 + lane * 2 < b) pair(q * 64 + lane * 2, first_r[q], first_i[q]);
            for (int k = AHEAD * 64 + lane * 2; k < b; k += 64)
                pair(k, *reinterpret_cast<const uint32_t*>(wr + k), *reinterpret_cast<const uint32_t*>(wi + k));
        } else {
            for (int k = lane; k < b; k += 32) {
                const float fr = to_f32(wr[k]), fi = to_f32(wi[k]);
#pragma unroll
                for (int tt = 0; tt < kLruTokens; ++tt) {
                    const float x = us[tt * b + k];
                    v[2 * tt] = fmaf(fr, x, v[2 * tt]);
                    v[2 * tt + 1] = fmaf(fi, x, v[2 * tt + 1]);
                }
            }
        }
#pragma unroll
        for (int half = kLruTokens, o = 16; half >= 1; half >>= 1, o >>= 1) {
            const bool upper = (lane & o) != 0;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float give = upper ? v[i] : v[i + half], keep = upper ? v[i + half] : v[i];
                v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
            }
        }
        v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);   // lane l: sum l / 2, that is token l / 4, Ra (even) or Ri (odd)
        const float zi = __shfl_down_sync(0xffffffffu, v[0], 2);
        if (finish) {
            const float2 p = lru_pair(v[0] + br, zi + bi, us[(lane >> 2) * b + col], rate);
            const float S = lru_apply(p.x, before, p.y);
            if (st) *st = S;
            out[(size_t)mine * C + c] = from_f32<T>(out_scale * S * gelu_tanhf_(gate + yb));
        }
    }
}

}  // namespace cib

using namespace cib;

// Rows may hold the gates of a bfloat16 engine in the tensor-core form: blocks of a multiple of 32 channels.
extern "C" int cib_lru_mma_supports(int b) { return b > 0 && b % kLK == 0; }

// One launch: u [tokens][>= C]; w [blocks][2 b][b] of u's type; bias float32 [2][C] (of Ra, then of Ri); sp = softplus(lam) float32
// [C]; pairs float32 [tokens][C][2] (see lru_pair).  logits null: the tensor-core form; else float32 [tokens][blocks][2 b], the products themselves.
extern "C" int cib_lru_gates(const void* u, int dtype, int u_stride, const void* w, const float* logits, const float* bias, const float* sp,
                             float* pairs, int C, int blocks, int num_tokens, cudaStream_t stream) {
    CIB_REQUIRE(C > 0 && blocks > 0 && C % blocks == 0 && u_stride >= C && num_tokens >= 0, "lru_gates: bad sizes");
    if (num_tokens == 0) return 0;
    const int b = C / blocks;
    if (!logits) {
        CIB_REQUIRE(dtype == kBF16 && cib_lru_mma_supports(b) && u_stride % 8 == 0 && (uintptr_t)u % 16 == 0, "lru_gates: the rows do not fit the tensor-core form");
        const int tiles = (b + kLN - 1) / kLN;
        CIB_REQUIRE((long long)blocks * tiles <= 65535, "lru_gates: too many blocks");
        launch_pdl(lru_gates_mma_kernel, dim3((num_tokens + kLM - 1) / kLM, blocks * tiles), dim3(128), 0, stream, prompt_pdl(),
                   (const __nv_bfloat16*)u, u_stride, (const __nv_bfloat16*)w, bias, sp, reinterpret_cast<float2*>(pairs), C, b, num_tokens);
    } else {
        const long long total = (long long)num_tokens * C;
        const unsigned grid = (unsigned)((total + 255) / 256);
        if (dtype == kF32) lru_gates_kernel<float><<<grid, 256, 0, stream>>>((const float*)u, u_stride, logits, bias, sp, reinterpret_cast<float2*>(pairs), C, b, total);
        else if (dtype == kBF16) lru_gates_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>((const __nv_bfloat16*)u, u_stride, logits, bias, sp, reinterpret_cast<float2*>(pairs), C, b, total);
        else CIB_REQUIRE(false, "lru_gates: bad dtype %d", dtype);
    }
    CIB_LAUNCH_CHECK("lru_gates");
    return 0;
}

// pairs float32 [tokens][C][2]; y rows `y_stride` apart, of out's type; state float32 [slots][C]; out [tokens][C].  longest: tokens of
// the longest request (or an upper bound), which chooses how many warps share a request's tokens.
extern "C" int cib_lru_scan(const float* pairs, const void* y, int dtype, int y_stride, const float* y_bias, float out_scale, float* state,
                            const int* query_start_loc, const int* state_slots, int num_slots, int num_requests, int longest, void* out, int C,
                            int num_tokens, cudaStream_t stream) {
    CIB_REQUIRE(C > 0 && y_stride >= C && num_requests >= 0 && num_requests <= 65535 && num_tokens >= 0, "lru_scan: bad sizes");
    if (num_tokens == 0 || num_requests == 0) return 0;
    int warps = 1;
    while (warps < kLruMaxWarps && warps * kLruUnroll < longest) warps <<= 1;
    const dim3 grid((C + 31) / 32, num_requests), block(32, warps);
    const bool pdl = prompt_pdl();
#define CIB_LRU(T)                                                                                                                       \
    launch_pdl(lru_scan_kernel<T>, grid, block, 0, stream, pdl, reinterpret_cast<const float2*>(pairs), (const T*)y, y_stride, y_bias,       \
               out_scale, state, query_start_loc, state_slots, num_slots, (T*)out, C)
    if (dtype == kF32) CIB_LRU(float);
    else if (dtype == kBF16) CIB_LRU(__nv_bfloat16);
    else CIB_REQUIRE(false, "lru_scan: bad dtype %d", dtype);
#undef CIB_LRU
    CIB_LAUNCH_CHECK("lru_scan");
    return 0;
}

extern "C" int cib_lru_decode(const void* u, int dtype, int u_stride, const void* w, const float* bias, const float* sp, const void* y,
                              int y_stride, const float* y_bias, float out_scale, float* state, const int* state_slots, int num_slots,
                              void* out, int C, int blocks, int num_tokens, cudaStream_t stream) {
    CIB_REQUIRE(C > 0 && blocks > 0 && C % blocks == 0 && u_stride >= C && y_stride >= C && num_tokens >= 0, "lru_decode: bad sizes");
    if (num_tokens == 0) return 0;
    const int b = C / blocks, per = kLruDecodeWarps;
    const size_t smem = (size_t)kLruTokens * b * sizeof(float);
    CIB_REQUIRE(smem <= 48 * 1024, "lru_decode: blocks of %d channels are beyond this kernel", b);
    const dim3 grid(blocks, (b + per - 1) / per);
    const bool pdl = prompt_pdl();
#define CIB_LRU(T, VEC)                                                                                                                  \
    launch_pdl(lru_decode_kernel<T, VEC>, grid, dim3(kLruDecodeWarps * 32), smem, stream, pdl, (const T*)u, u_stride, (const T*)w, bias, sp, \
               (const T*)y, y_stride, y_bias, out_scale, state, state_slots, num_slots, (T*)out, C, b, num_tokens)
    if (dtype == kF32) CIB_LRU(float, false);
    else if (dtype == kBF16 && b % 2 == 0 && (uintptr_t)w % 4 == 0) CIB_LRU(__nv_bfloat16, true);
    else if (dtype == kBF16) CIB_LRU(__nv_bfloat16, false);
    else CIB_REQUIRE(false, "lru_decode: bad dtype %d", dtype);
#undef CIB_LRU
    CIB_LAUNCH_CHECK("lru_decode");
    return 0;
}
