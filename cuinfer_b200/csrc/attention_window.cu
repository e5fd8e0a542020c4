// Grouped-query attention whose keys and values have sizes of their own, with a capped score and a window that keeps
// the first tokens of a sequence visible: the step before the attention (biases, norm, rotation, query temperature, value
// mixing, cache write) and the plain all-sizes attention kernel (a warp per query token and head), which is the 32-bit
// path.  Every step is optional, so that one pair of kernels serves several kinds of attention layer.
//
// Per token and head, with the query q and key k of d values and the value v of dv values:
//   q, k, v += their biases (32-bit);
//   with `taps`, q, k and v each pass a short causal convolution over time per channel (biases included in its input; the
//   inputs before the step's rows come from the request's state, zeros before the start of a sequence); the queries
//   then go to rows of their own, since other tokens still read the projected ones;
//   with `q_only` the rows hold queries only: keys and values are those another layer has cached;
//   with `value_from_key` there is no v in the rows: v = k as it stands here, before norm and rotation;
//   rotation of the first `rot_dims` values by the angle pos * freq[i] (32-bit angle, full-range sine and cosine, both
//   multiplied by `rot_gain`), in neighbouring pairs (2i, 2i+1) or in halves (i, i + rot_dims / 2);
//   q and k divided by their root mean square (eps inside the root) and multiplied by a gain of d values shared by all
//   heads (null: no gain), after the rotation or, with `norm_first`, before it; with `norm_rows` one root mean square over
//   all of a token's query heads (and one over its key heads) with a gain per value of the row;
//   q multiplied by the query temperature 1 + coef * ln(floor((pos + 1) / every) + 1);
//   v = (1 - lambda) * v + lambda * v_first for a layer that mixes in an earlier layer's values of the same token;
//   score = scale * q.k, then cap * tanh(score / cap) if cap > 0, then minus slope[head] * (i - j) (a distance bias) or
//   minus r1[head] * ln(1 + r2[head] * (i - j)) (one that grows with the logarithm of the distance);
//   query at position i sees key j when j <= i and (window == 0 or i - j < window or j < keep_first); with `chunked`
//   the window is a chunk instead: j >= floor(i / window) * window;
//   softmax over the visible keys, whose denominator also holds exp(sink[head]) when sinks are given (a sink has no key
//   and no value and is neither scaled nor biased); weighted sum of the values; with `sigmoid_bias` nothing is
//   normalised: a key counts with sigmoid(score + sigmoid_bias[head]);
//   with `gate` the result is multiplied by sigmoid of the token's gate logit, one per value or one per head.
// Everything after the loads is 32-bit; exponentials, tangents, sines, logarithms are the exact ones.
//
// Cache layout of one layer run: [page][kv head][slot in page][d + dv] — a token's key and value side by side.
#include "mma_utils.cuh"

namespace cib {

constexpr int kPrepWarps = 8;
constexpr int kPrepMaxPairsPerLane = 8;      // d and dv up to 512

// What the step before the attention does beside rotation and cache write; every pointer may be null.
struct PrepOptions {
    const float* bias;        // [H*d + G*d + G*dv] added to the packed rows
    const float* q_gain;      // [d] gain of the query heads' norm
    const float* k_gain;      // [d] gain of the key heads' norm
    int norm;                 // 0: no norm of q and k; 1: divided by their root mean square (times the gain, if any)
    int norm_first;           // the norm comes before the rotation
    int rot_half;             // rotation pairs are (i, i + rot_dims / 2) instead of (2i, 2i + 1)
    int has_temp;             // queries are multiplied by 1 + temp_coef * ln(floor((pos + 1) / temp_every) + 1)
    float temp_coef;
    int temp_every;
    int value_from_key;       // the packed rows are [q | k]: a token's value is its key as it stands before norm and rotation
    float rot_gain;           // cosine and sine are both multiplied by this (1: a pure rotation)
    int q_only;               // the packed rows are queries only; nothing is cached
    // short causal convolution; taps null: none
    const float* taps;        // [taps_n][columns], the last row is the current token's
    int taps_n;
    float* conv_state;        // [slots][taps_n - 1][columns], oldest first
    const int* query_start_loc;
    const int* token_request;
    const int* state_slots;
    int num_state_slots;
    int conv_update;          // every request brings one token: the lane that reads a channel's state also moves it on
    int norm_rows;            // the norm is over all query heads (all key heads) of a token; the gains have a value per column
};

// The conv of one column of one token's row (see PrepOptions): u_t = x_t + bias; y = sum_j taps[j] u_(t - taps_n + 1 + j).
template <typename T>
__device__ __forceinline__ float conv_column(const T* __restrict__ rows, int stride, int t, int start, float* __restrict__ state,
                                             int columns, int col, const PrepOptions& opt) {
    const float b = opt.bias ? opt.bias[col] : 0.f;
    const int K = opt.taps_n;
    const float u = to_f32(rows[(size_t)t * stride + col]) + b;
    float y = opt.taps[(size_t)(K - 1) * columns + col] * u;
    for (int jb = 1; jb < K; ++jb) {                      // jb tokens back
        const int tt = t - jb;
        float x = 0.f;
        if (tt >= start) x = to_f32(rows[(size_t)tt * stride + col]) + b;
        else if (state) x = state[(size_t)(K - 1 - (start - tt)) * columns + col];
        y = fmaf(opt.taps[(size_t)(K - 1 - jb) * columns + col], x, y);
    }
    if (opt.conv_update && state) {
        for (int i = 0; i + 2 < K; ++i) state[(size_t)i * columns + col] = state[(size_t)(i + 1) * columns + col];
        if (K > 1) state[(size_t)(K - 2) * columns + col] = u;
    }
    return y;
}

// One warp per (token, vector): H query heads, G key heads, G value heads of the packed rows [q | k | v] (with
// `value_from_key` there are no value vectors: the key's warp stores the value too).  C: pairs of values a lane holds
// (d <= 64 C).
// row_factor: with `norm_rows`, one over the root mean square of the token's queries or keys.
template <typename T, int C>
__device__ __forceinline__ void
prep_vector(int t, int vec, float row_factor, T* qkv, int stride, T* q_out, int q_out_stride, const int* __restrict__ positions,
            const int* __restrict__ slot_mapping, const float* __restrict__ freq, int rot_dims, float eps,
            int H, int G, int d, int dv, const T* __restrict__ v_first, int v_first_stride,
            AnyVec lambda, int has_lambda, T* __restrict__ cache, long long num_slots, int page_size, const PrepOptions& opt) {
    const int lane = threadIdx.x & 31;
    T* row = qkv + (size_t)t * stride;
    const int slot = slot_mapping ? slot_mapping[t] : -1;
    const bool store = cache && slot >= 0 && slot < num_slots;
    const int width = d + dv;
    const int columns = opt.q_only ? H * d : (H + G) * d + (opt.value_from_key ? 0 : G * dv);
    int start = 0;
    float* state = nullptr;
    if (opt.taps) {
        const int r = opt.token_request[t];
        start = opt.query_start_loc[r];
        const int ss = opt.state_slots[r];
        if (opt.taps_n > 1 && ss >= 0 && ss < opt.num_state_slots) state = opt.conv_state + (size_t)ss * (opt.taps_n - 1) * columns;
    }
    if (vec >= H + G) {                                   // a value head: bias, convolution, mix and store
        const int g = vec - H - G;
        if (!store && !(opt.taps && opt.conv_update)) return;
        const size_t off = (size_t)H * d + (size_t)G * d + (size_t)g * dv;
        const T* v = row + off;
        const float lam = has_lambda ? lambda[0] : 0.f;
        T* dst = store ? cache + (((size_t)(slot / page_size) * G + g) * page_size + slot % page_size) * width + d : nullptr;
        for (int i = lane; i < dv; i += 32) {
            float x;
            if (opt.taps) {
                x = conv_column(qkv, stride, t, start, state, columns, (int)off + i, opt);
                if (!store) continue;
            } else {
                x = to_f32(v[i]);
                if (opt.bias) x += opt.bias[off + i];
            }
            if (has_lambda) x = (1.f - lam) * x + lam * to_f32(v_first[(size_t)t * v_first_stride + (size_t)g * dv + i]);
            dst[i] = from_f32<T>(x);
        }
        return;
    }
    const bool is_key = vec >= H;
    const size_t off = is_key ? (size_t)H * d + (size_t)(vec - H) * d : (size_t)vec * d;
    T* x = row + off;
    const float* bias = opt.bias ? opt.bias + off : nullptr;
    const float* gain = is_key ? opt.k_gain : opt.q_gain;
    if (gain && opt.norm_rows) gain += is_key ? (size_t)(vec - H) * d : off;
    const int ipos = positions[t];
    const float pos = (float)ipos;
    const int half = rot_dims / 2;
    float a[C], b[C];
    // pair p of the lane's pairs: the rotation partners, or two neighbours of the part that is not rotated
    auto first_of = [&](int p) { return opt.rot_half && p < half ? p : 2 * p; };
    auto second_of = [&](int p) { return opt.rot_half && p < half ? p + half : 2 * p + 1; };
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int p = c * 32 + lane, e0 = first_of(p), e1 = second_of(p);
        if (opt.taps) {
            a[c] = e0 < d ? conv_column(qkv, stride, t, start, state, columns, (int)off + e0, opt) : 0.f;
            b[c] = e1 < d ? conv_column(qkv, stride, t, start, state, columns, (int)off + e1, opt) : 0.f;
        } else {
            a[c] = e0 < d ? to_f32(x[e0]) + (bias ? bias[e0] : 0.f) : 0.f;
            b[c] = e1 < d ? to_f32(x[e1]) + (bias ? bias[e1] : 0.f) : 0.f;
        }
    }
    if (opt.value_from_key && is_key && store) {          // dv == d: the value is the key as projected
        T* vdst = cache + (((size_t)(slot / page_size) * G + (vec - H)) * page_size + slot % page_size) * width + d;
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const int p = c * 32 + lane, e0 = first_of(p), e1 = second_of(p);
            if (e0 < d) vdst[e0] = from_f32<T>(a[c]);
            if (e1 < d) vdst[e1] = from_f32<T>(b[c]);
        }
    }
    auto normalise = [&]() {
        float factor = row_factor;
        if (!opt.norm_rows) {
            float ss = 0.f;
#pragma unroll
            for (int c = 0; c < C; ++c) ss += a[c] * a[c] + b[c] * b[c];
            ss = warp_sum(ss);
            factor = 1.f / sqrtf(ss / (float)d + eps);
        }
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const int p = c * 32 + lane, e0 = first_of(p), e1 = second_of(p);
            a[c] *= factor * (gain && e0 < d ? gain[e0] : 1.f);
            b[c] *= factor * (gain && e1 < d ? gain[e1] : 1.f);
        }
    };
    if (opt.norm && opt.norm_first) normalise();
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int p = c * 32 + lane;
        if (p < half && second_of(p) < d) {
            float sn, cs;
            sincosf(pos * freq[p], &sn, &cs);
            sn *= opt.rot_gain;
            cs *= opt.rot_gain;
            const float u = a[c], v = b[c];
            a[c] = u * cs - v * sn;
            b[c] = v * cs + u * sn;
        }
    }
    if (opt.norm && !opt.norm_first) normalise();
    if (opt.has_temp && !is_key) {
        const float temp = 1.f + opt.temp_coef * logf((float)((ipos + 1) / opt.temp_every + 1));
#pragma unroll
        for (int c = 0; c < C; ++c) { a[c] *= temp; b[c] *= temp; }
    }
    T* dst = q_out ? q_out + (size_t)t * q_out_stride + off : x;
    if (is_key) {
        if (!store) return;
        dst = cache + (((size_t)(slot / page_size) * G + (vec - H)) * page_size + slot % page_size) * width;
    }
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int p = c * 32 + lane, e0 = first_of(p), e1 = second_of(p);
        if (e0 < d) dst[e0] = from_f32<T>(a[c]);
        if (e1 < d) dst[e1] = from_f32<T>(b[c]);
    }
}

template <typename T, int C>
__global__ void __launch_bounds__(kPrepWarps * 32)
window_attention_prep_kernel(T* qkv, int stride, T* q_out, int q_out_stride, const int* __restrict__ positions,
                             const int* __restrict__ slot_mapping, const float* __restrict__ freq, int rot_dims, float eps,
                             int H, int G, int d, int dv, const T* __restrict__ v_first, int v_first_stride,
                             AnyVec lambda, int has_lambda, T* __restrict__ cache, long long num_slots, int page_size,
                             int num_tokens, PrepOptions opt) {
    const int vectors = opt.q_only ? H : opt.value_from_key ? H + G : H + 2 * G;
    const long long w = (long long)blockIdx.x * kPrepWarps + (threadIdx.x >> 5);
    if (w >= (long long)num_tokens * vectors) return;
    prep_vector<T, C>((int)(w / vectors), (int)(w % vectors), 1.f, qkv, stride, q_out, q_out_stride, positions, slot_mapping, freq, rot_dims,
                      eps, H, G, d, dv, v_first, v_first_stride, lambda, has_lambda, cache, num_slots, page_size, opt);
}

// The norm over whole rows of queries and keys: a block per token sums both rows' squares (biases included), then its warps
// take the vectors one by one.  PLAIN (bfloat16, sizes in multiples of 8, no bias, rotation or temperature): eight values a
// lane, the rows staged in registers between the two passes where they fit.
template <typename T, int C, bool PLAIN>
__global__ void __launch_bounds__(kPrepWarps * 32)
window_attention_prep_rows_kernel(T* qkv, int stride, const int* __restrict__ positions, const int* __restrict__ slot_mapping,
                                  const float* __restrict__ freq, int rot_dims, float eps, int H, int G, int d, int dv,
                                  T* __restrict__ cache, long long num_slots, int page_size, PrepOptions opt) {
    __shared__ float scratch[33];
    const int t = blockIdx.x;
    T* row = qkv + (size_t)t * stride;
    const int nq = H * d, nk = opt.q_only ? 0 : G * d;
    griddep_launch();
    griddep_wait();
    if constexpr (PLAIN) {
        constexpr int CH = 4;                             // rows of up to 8 192 values stay in registers
        const int total = nq + nk;
        uint4 held[CH];
        float sq = 0.f, sk = 0.f;
        auto add = [&](const uint4& v, int i) {
            const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
            float s = 0.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 f = __bfloat1622float2(h[e]);
                s = fmaf(f.x, f.x, fmaf(f.y, f.y, s));
            }
            if (i < nq) sq += s; else sk += s;
        };
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            const int i = (c * kPrepWarps * 32 + threadIdx.x) * 8;
            if (i < total) held[c] = *reinterpret_cast<const uint4*>(row + i);
        }
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            const int i = (c * kPrepWarps * 32 + threadIdx.x) * 8;
            if (i < total) add(held[c], i);
        }
        for (int i = (CH * kPrepWarps * 32 + threadIdx.x) * 8; i < total; i += kPrepWarps * 32 * 8) add(*reinterpret_cast<const uint4*>(row + i), i);
        sq = block_sum(sq, scratch);
        sk = block_sum(sk, scratch);
        const float fq = 1.f / sqrtf(sq / (float)nq + eps), fk = nk ? 1.f / sqrtf(sk / (float)nk + eps) : 0.f;
        const int slot = slot_mapping ? slot_mapping[t] : -1;
        const bool store = cache && slot >= 0 && slot < num_slots;
        const int width = d + dv;
        T* page = store ? cache + ((size_t)(slot / page_size) * G * page_size + slot % page_size) * width : nullptr;
        auto place = [&](uint4 v, int i) {
            const bool key = i >= nq;
            if (key && !store) return;
            const int at = key ? i - nq : i;
            const float f = key ? fk : fq;
            const float* gain = key ? opt.k_gain : opt.q_gain;
            uint32_t* p = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 x = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&v)[e]);
                const float2 g = gain ? *reinterpret_cast<const float2*>(gain + at + 2 * e) : make_float2(1.f, 1.f);
                __nv_bfloat162 y = __floats2bfloat162_rn(x.x * f * g.x, x.y * f * g.y);
                p[e] = *reinterpret_cast<uint32_t*>(&y);
            }
            T* dst = key ? page + (size_t)(at / d) * page_size * width + at % d : row + i;
            *reinterpret_cast<uint4*>(dst) = v;
        };
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            const int i = (c * kPrepWarps * 32 + threadIdx.x) * 8;
            if (i < total) place(held[c], i);
        }
        for (int i = (CH * kPrepWarps * 32 + threadIdx.x) * 8; i < total; i += kPrepWarps * 32 * 8) place(*reinterpret_cast<const uint4*>(row + i), i);
        if (!store || opt.q_only) return;
        for (int i = threadIdx.x * 8; i < G * dv; i += kPrepWarps * 32 * 8)
            *reinterpret_cast<uint4*>(page + (size_t)(i / dv) * page_size * width + d + i % dv) = *reinterpret_cast<const uint4*>(row + total + i);
    } else {
        float sq = 0.f, sk = 0.f;
        for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
            const float x = to_f32(row[i]) + (opt.bias ? opt.bias[i] : 0.f);
            if (i < nq) sq = fmaf(x, x, sq); else sk = fmaf(x, x, sk);
        }
        sq = block_sum(sq, scratch);
        sk = block_sum(sk, scratch);                      // also: every square is in before a query is rewritten
        const float fq = 1.f / sqrtf(sq / (float)nq + eps), fk = nk ? 1.f / sqrtf(sk / (float)nk + eps) : 0.f;
        const int vectors = opt.q_only ? H : H + 2 * G;
        for (int vec = threadIdx.x >> 5; vec < vectors; vec += kPrepWarps)
            prep_vector<T, C>(t, vec, vec < H ? fq : fk, qkv, stride, nullptr, 0, positions, slot_mapping, freq, rot_dims, eps, H, G, d, dv,
                              nullptr, 0, AnyVec{nullptr, 0}, 0, cache, num_slots, page_size, opt);
    }
}

constexpr int kWinWarps = 4;
constexpr int kWinMaxAcc = 16;               // dv up to 512

template <typename T>
__global__ void __launch_bounds__(kWinWarps * 32)
window_attention_generic_kernel(const T* __restrict__ q, int q_stride, T* __restrict__ out, int out_stride,
                                const T* __restrict__ cache, int num_pages, int page_size,
                                const int* __restrict__ block_table, int table_stride, const int* __restrict__ positions,
                                const int* __restrict__ token_request, int H, int G, int d, int dv, float scale, float cap,
                                int window, int keep_first, int chunked, const float* __restrict__ slopes,
                                const float* __restrict__ sinks, const float* __restrict__ sigmoid_bias,
                                const float* __restrict__ r1, const float* __restrict__ r2, const T* __restrict__ gate,
                                int gate_stride, int gate_per_head) {
    extern __shared__ float smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x;
    const int head = blockIdx.y * kWinWarps + warp;
    if (head >= H) return;
    const int g = head / (H / G);
    float* qs = smem + warp * d;
    const int r = token_request[t];
    const int pos = positions[t];
    const int lo = window > 0 ? (chunked ? pos / window * window : max(0, pos - window + 1)) : 0;
    const float slope = slopes ? slopes[head] : 0.f;
    const float log_a = r1 ? r1[head] : 0.f, log_b = r1 ? r2[head] : 0.f;
    const float pb = sigmoid_bias ? sigmoid_bias[head] : 0.f;
    const int kept = window > 0 ? min(keep_first, lo) : 0;        // keys 0..kept-1 lie before the window and stay visible
    const int* table = block_table + (size_t)r * table_stride;
    const T* qp = q + (size_t)t * q_stride + (size_t)head * d;
    for (int i = lane; i < d; i += 32) qs[i] = to_f32(qp[i]);
    __syncwarp();

    float acc[kWinMaxAcc];
#pragma unroll
    for (int k = 0; k < kWinMaxAcc; ++k) acc[k] = 0.f;
    float m = -INFINITY, l = 0.f;
    const int width = d + dv;
    const float inv_cap = cap > 0.f ? 1.f / cap : 0.f;

    for (int seg = 0; seg < 2; ++seg) {
        const int begin = seg == 0 ? 0 : lo, end = seg == 0 ? kept : pos + 1;
        for (int c = begin; c < end; c += 32) {
            const int j = c + lane;
            float s = -INFINITY;
            const T* row = nullptr;
            if (j < end) {
                const int page = table[j / page_size];
                if (page >= 0 && page < num_pages) {
                    row = cache + (((size_t)page * G + g) * page_size + j % page_size) * width;
                    float dot = 0.f;
                    for (int i = 0; i < d; ++i) dot = fmaf(qs[i], to_f32(row[i]), dot);
                    s = dot * scale;
                    if (cap > 0.f) s = cap * tanhf(s * inv_cap);
                    s -= slope * (float)(pos - j);
                    if (r1) s -= log_a * log1pf(log_b * (float)(pos - j));
                }
            }
            float p;
            if (sigmoid_bias) {                                   // weights of their own, nothing to rescale
                p = s == -INFINITY ? 0.f : 1.f / (1.f + expf(-(s + pb)));
            } else {
                const float m_new = fmaxf(m, warp_max(s));
                if (m_new == -INFINITY) continue;                 // nothing visible in this chunk
                p = s == -INFINITY ? 0.f : expf(s - m_new);
                const float corr = m == -INFINITY ? 0.f : expf(m - m_new);
                l = l * corr + warp_sum(p);
                m = m_new;
#pragma unroll
                for (int k = 0; k < kWinMaxAcc; ++k) acc[k] *= corr;
            }
            const int count = min(32, end - c);
            for (int jj = 0; jj < count; ++jj) {
                const float pj = __shfl_sync(0xffffffffu, p, jj);
                const T* vj = reinterpret_cast<const T*>(__shfl_sync(0xffffffffu, reinterpret_cast<uintptr_t>(row), jj));
                if (pj == 0.f || vj == nullptr) continue;
#pragma unroll
                for (int k = 0; k < kWinMaxAcc; ++k) {
                    const int i = k * 32 + lane;
                    if (i < dv) acc[k] = fmaf(pj, to_f32(vj[d + i]), acc[k]);
                }
            }
        }
    }
    if (sinks) {                                                  // the sink joins the denominator and nothing else
        const float sink = sinks[head];
        const float m_new = fmaxf(m, sink);
        const float corr = m == -INFINITY ? 0.f : expf(m - m_new);
        l = l * corr + expf(sink - m_new);
#pragma unroll
        for (int k = 0; k < kWinMaxAcc; ++k) acc[k] *= corr;
    }
    float inv = sigmoid_bias ? 1.f : l > 0.f ? 1.f / l : 0.f;
    T* op = out + (size_t)t * out_stride + (size_t)head * dv;
    const T* gp = gate ? gate + (size_t)t * gate_stride + (gate_per_head ? head : head * dv) : nullptr;
    if (gp && gate_per_head) inv *= 1.f / (1.f + expf(-to_f32(gp[0])));
#pragma unroll
    for (int k = 0; k < kWinMaxAcc; ++k) {
        const int i = k * 32 + lane;
        if (i < dv) {
            float y = acc[k] * inv;
            if (gp && !gate_per_head) y *= 1.f / (1.f + expf(-to_f32(gp[i])));
            op[i] = from_f32<T>(y);
        }
    }
}

}  // namespace cib

using namespace cib;

// bias (float32 [H*d + G*d + G*dv]), q_gain / k_gain (float32 [d]) may be null.  norm: 0 none, 1 root mean square (with
// the gains, if given); norm_first: before the rotation; rot_half: pairs (i, i + rot_dims / 2); has_temp: the query
// temperature with temp_coef and temp_every; value_from_key: rows are [q | k] and a token's cached value is its key before
// norm and rotation (dv == d); rot_gain: a factor on both cosine and sine.  q_out: where the queries go (null: back into
// the rows; must be given with taps).  q_only: rows are [q].  taps (float32 [taps_n][columns], null: none): the short
// convolution, whose state conv_state [slots][taps_n - 1][columns] is only read here unless conv_update says that every
// request brings one token (else cib_conv_state_update follows).
extern "C" int cib_window_attention_prep(void* qkv, int dtype, int stride, void* q_out, int q_out_stride, const int* positions, const int* slot_mapping,
                                         const float* freq, int rot_dims, float eps, int H, int G, int d, int dv,
                                         const void* v_first, int v_first_stride, const void* lambda, int lambda_dtype,
                                         void* cache, long long num_slots, int page_size, int num_tokens,
                                         const float* bias, const float* q_gain, const float* k_gain, int norm, int norm_first,
                                         int rot_half, int has_temp, float temp_coef, int temp_every, int value_from_key,
                                         float rot_gain, int q_only, const float* taps, int taps_n, float* conv_state,
                                         const int* query_start_loc, const int* token_request, const int* state_slots,
                                         int num_state_slots, int conv_update, int norm_rows, cudaStream_t stream) {
    CIB_REQUIRE(!norm_rows || (norm && !taps && !value_from_key && !v_first && !q_out),
                "window_attention_prep: a norm over whole rows beside a convolution, mixed values or values taken from keys is not built");
    CIB_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0, "window_attention_prep: bad head counts or sizes");
    CIB_REQUIRE(!taps || (taps_n >= 1 && q_out && (taps_n == 1 || conv_state) && query_start_loc && token_request && state_slots),
                "window_attention_prep: a convolution needs its state, the requests' bounds and a place for the queries");
    CIB_REQUIRE(!q_only || (!value_from_key && v_first == nullptr), "window_attention_prep: rows of queries hold no values");
    CIB_REQUIRE(!(taps && (value_from_key || v_first)), "window_attention_prep: a convolution beside values taken from keys or mixed values is not built");
    CIB_REQUIRE(d <= 64 * kPrepMaxPairsPerLane, "window_attention_prep: head size %d is beyond %d", d, 64 * kPrepMaxPairsPerLane);
    CIB_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= d && (rot_dims == 0 || freq), "window_attention_prep: bad rotation");
    CIB_REQUIRE((v_first == nullptr) == (lambda == nullptr), "window_attention_prep: mixing needs both the values and the factor");
    CIB_REQUIRE(!has_temp || temp_every > 0, "window_attention_prep: the query temperature needs a positive period");
    CIB_REQUIRE(!value_from_key || (d == dv && v_first == nullptr), "window_attention_prep: values taken from the keys have the keys' size and are not mixed");
    if (num_tokens == 0) return 0;
    const long long warps = (long long)num_tokens * (q_only ? H : value_from_key ? H + G : H + 2 * G);
    const int blocks = (int)((warps + kPrepWarps - 1) / kPrepWarps);
    AnyVec lam{lambda, lambda_dtype == kBF16};
    PrepOptions opt{bias, q_gain, k_gain, norm, norm_first, rot_half, has_temp, temp_coef, temp_every, value_from_key, rot_gain, q_only,
                    taps, taps_n, conv_state, query_start_loc, token_request, state_slots, num_state_slots, conv_update, norm_rows};
    if (norm_rows) {
        const bool pdl = prompt_pdl();
        auto gain_ok = [](const float* g) { return (uintptr_t)g % 8 == 0; };
        const bool plain = dtype == kBF16 && d % 8 == 0 && dv % 8 == 0 && stride % 8 == 0 && !bias && !rot_dims && !has_temp &&
                           (uintptr_t)qkv % 16 == 0 && (uintptr_t)cache % 16 == 0 && gain_ok(q_gain) && gain_ok(k_gain);
#define CIB_PREP_ROWS(T, C, PLAIN)                                                                                            \
    launch_pdl(window_attention_prep_rows_kernel<T, C, PLAIN>, dim3(num_tokens), dim3(kPrepWarps * 32), 0, stream, pdl, (T*)qkv, stride,  \
               positions, slot_mapping, freq, rot_dims, eps, H, G, d, dv, (T*)cache, num_slots, page_size, opt)
        if (plain) CIB_PREP_ROWS(__nv_bfloat16, 1, true);
        else if (dtype == kF32) { if (d <= 64) CIB_PREP_ROWS(float, 1, false); else if (d <= 128) CIB_PREP_ROWS(float, 2, false); else CIB_PREP_ROWS(float, 8, false); }
        else if (dtype == kBF16) { if (d <= 64) CIB_PREP_ROWS(__nv_bfloat16, 1, false); else if (d <= 128) CIB_PREP_ROWS(__nv_bfloat16, 2, false); else CIB_PREP_ROWS(__nv_bfloat16, 8, false); }
        else CIB_REQUIRE(false, "window_attention_prep: bad dtype %d", dtype);
#undef CIB_PREP_ROWS
        CIB_LAUNCH_CHECK("window_attention_prep");
        return 0;
    }
#define CIB_PREP(T, C)                                                                                                        \
    window_attention_prep_kernel<T, C><<<blocks, kPrepWarps * 32, 0, stream>>>(                                               \
        (T*)qkv, stride, (T*)q_out, q_out_stride, positions, slot_mapping, freq, rot_dims, eps, H, G, d, dv, (const T*)v_first, v_first_stride, lam,    \
        lambda != nullptr, (T*)cache, num_slots, page_size, num_tokens, opt)
#define CIB_PREP_BY_SIZE(T)                                                                                                   \
    {                                                                                                                         \
        if (d <= 64) CIB_PREP(T, 1);                                                                                          \
        else if (d <= 128) CIB_PREP(T, 2);                                                                                    \
        else if (d <= 256) CIB_PREP(T, 4);                                                                                    \
        else CIB_PREP(T, 8);                                                                                                  \
    }
    if (dtype == kF32) CIB_PREP_BY_SIZE(float)
    else if (dtype == kBF16) CIB_PREP_BY_SIZE(__nv_bfloat16)
    else CIB_REQUIRE(false, "window_attention_prep: bad dtype %d", dtype);
#undef CIB_PREP_BY_SIZE
#undef CIB_PREP
    CIB_LAUNCH_CHECK("window_attention_prep");
    return 0;
}

extern "C" int cib_window_attention_generic(const void* q, int dtype, int q_stride, void* out, int out_stride, const void* cache,
                                            int num_pages, int page_size, const int* block_table, int table_stride,
                                            const int* positions, const int* token_request, int num_tokens, int H, int G,
                                            int d, int dv, float scale, float cap, int window, int keep_first, int chunked,
                                            const float* slopes, const float* sinks, const float* sigmoid_bias, const float* r1,
                                            const float* r2, const void* gate, int gate_stride, int gate_per_head,
                                            cudaStream_t stream) {
    CIB_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0, "window_attention: bad head counts or sizes");
    CIB_REQUIRE((r1 == nullptr) == (r2 == nullptr), "window_attention: the logarithmic distance bias has two numbers per head");
    CIB_REQUIRE(!(sigmoid_bias && sinks), "window_attention: weights that are not normalised have no sink");
    CIB_REQUIRE(dv <= 32 * kWinMaxAcc, "window_attention: value size %d is beyond %d", dv, 32 * kWinMaxAcc);
    CIB_REQUIRE(d <= 2048, "window_attention: head size %d is beyond 2048", d);
    CIB_REQUIRE(window >= 0 && keep_first >= 0, "window_attention: bad window");
    if (num_tokens == 0) return 0;
    dim3 grid(num_tokens, (H + kWinWarps - 1) / kWinWarps);
    const size_t smem = (size_t)kWinWarps * d * sizeof(float);
    if (dtype == kF32)
        window_attention_generic_kernel<float><<<grid, kWinWarps * 32, smem, stream>>>((const float*)q, q_stride, (float*)out, out_stride, (const float*)cache, num_pages, page_size, block_table, table_stride, positions, token_request, H, G, d, dv, scale, cap, window, keep_first, chunked, slopes, sinks, sigmoid_bias, r1, r2, (const float*)gate, gate_stride, gate_per_head);
    else if (dtype == kBF16)
        window_attention_generic_kernel<__nv_bfloat16><<<grid, kWinWarps * 32, smem, stream>>>((const __nv_bfloat16*)q, q_stride, (__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)cache, num_pages, page_size, block_table, table_stride, positions, token_request, H, G, d, dv, scale, cap, window, keep_first, chunked, slopes, sinks, sigmoid_bias, r1, r2, (const __nv_bfloat16*)gate, gate_stride, gate_per_head);
    else
        CIB_REQUIRE(false, "window_attention: bad dtype %d", dtype);
    CIB_LAUNCH_CHECK("window_attention_generic");
    return 0;
}
