// Row-wise kernels around the matrix products: embedding gather, residual-add + RMSNorm,
// gather of the rows whose logits are wanted, and the SiLU-gated product.
//
// At the end: the scaled sum of two deltas with an RMS norm in groups, half the sum of two normed rows, tanh.
//
// Reference counterparts: csrc/ops/embedding.cu:18-36, csrc/ops/rms_norm.cu:18-73,
// csrc/ops/residual_rms_norm_fused.cu:26-110, csrc/ops/residual_add.cu:23-82, csrc/ops/swiglu.cu:34-60.
// Unlike those, every size is a run-time parameter, the residual stream is kept in 32 bits, and the
// add, the norm and the store of the new residual are one pass over the row.
#include <algorithm>

#include "common.cuh"
#include "mma_utils.cuh"

namespace cib {

template <typename T, int V> struct Vec;
template <> struct Vec<float, 4> {
    static __device__ __forceinline__ void load(const float* p, float* v) {
        float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
    static __device__ __forceinline__ void store(float* p, const float* v) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
};
template <> struct Vec<__nv_bfloat16, 4> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* v) {
        uint2 t = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&t.x);
        const __nv_bfloat162 b = *reinterpret_cast<const __nv_bfloat162*>(&t.y);
        v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]);
        __nv_bfloat162 b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 t;
        t.x = *reinterpret_cast<uint32_t*>(&a);
        t.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = t;
    }
};
template <typename T> struct Vec<T, 1> {
    static __device__ __forceinline__ void load(const T* p, float* v) { v[0] = to_f32(*p); }
    static __device__ __forceinline__ void store(T* p, const float* v) { *p = from_f32<T>(v[0]); }
};

// ---- embedding ---------------------------------------------------------------------------------
// out[t, :] = table[ids[t], :] * scale as 32-bit residual rows (the product is taken in 32 bits); an id outside the
// table gives a zero row and raises the flag (the host rejects such ids before they get here).
template <typename T, int V>
__global__ void embedding_gather_kernel(const int* __restrict__ ids, const T* __restrict__ table,
                                        float* __restrict__ out, int hidden, int vocab,
                                        int* __restrict__ bad_flag, float scale, int copies) {
    const int t = blockIdx.x;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0 && bad_flag) atomicExch(bad_flag, 1);
    const T* src = table + (size_t)(ok ? id : 0) * hidden;
    float* dst = out + (size_t)t * copies * hidden;        // a residual of several streams starts with every stream equal
    for (int i = threadIdx.x * V; i < hidden; i += blockDim.x * V) {
        float v[V];
        Vec<T, V>::load(src + i, v);
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = ok ? v[k] * scale : 0.f;
        for (int c = 0; c < copies; ++c) Vec<float, V>::store(dst + (size_t)c * hidden + i, v);
    }
}

// ---- residual add + RMSNorm ---------------------------------------------------------------------
// x = residual (+ delta); residual = x (when a delta is given); out = x * rsqrt(mean(x^2) + eps) * w.
// Squares, mean, rsqrt and the product are 32-bit; the output is rounded once.
template <typename TD, typename TO, int V>
__global__ void add_rmsnorm_kernel(float* __restrict__ residual, const TD* __restrict__ delta,
                                   AnyVec weight, float eps, TO* __restrict__ out, int hidden) {
    __shared__ float scratch[33];
    const size_t row = (size_t)blockIdx.x * hidden;
    float* res = residual + row;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < hidden; i += blockDim.x * V) {
        float x[V];
        Vec<float, V>::load(res + i, x);
        if (delta) {
            float d[V];
            Vec<TD, V>::load(delta + row + i, d);
#pragma unroll
            for (int k = 0; k < V; ++k) x[k] += d[k];
            Vec<float, V>::store(res + i, x);
        }
#pragma unroll
        for (int k = 0; k < V; ++k) ss += x[k] * x[k];
    }
    ss = block_sum(ss, scratch);
    const float factor = rsqrtf(ss / (float)hidden + eps);
    if (!out) return;
    for (int i = threadIdx.x * V; i < hidden; i += blockDim.x * V) {
        float x[V];
        Vec<float, V>::load(res + i, x);   // this thread wrote exactly these elements above
#pragma unroll
        for (int k = 0; k < V; ++k) x[k] = x[k] * factor * weight[i + k];
        Vec<TO, V>::store(out + row + i, x);
    }
}

// Many rows (prompt portions): a warp per row, the whole row in registers (CH chunks of four values per lane), every
// load issued before the first use, one shuffle reduction, no second read of the residual.  Same arithmetic and the
// same order of operations per element as the kernel above; only the order of the sum of squares differs.
template <typename TD, typename TO, int CH>
__global__ void __launch_bounds__(256)
add_rmsnorm_rows_kernel(float* __restrict__ residual, const TD* __restrict__ delta, AnyVec weight, float eps,
                        TO* __restrict__ out, int hidden, int rows) {
    // the gains do not come from the kernel before this one: they are in shared memory before the dependency wait,
    // instead of a trip to the L2 after the reduction
    __shared__ __align__(16) float s_gain[CH * 128];
    griddep_launch();
    if (out)
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) s_gain[i] = weight[i];
    griddep_wait();          // residual and delta come from the kernels before this one
    __syncthreads();
    const int lane = threadIdx.x & 31;
    const int r = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (r >= rows) return;
    const size_t row = (size_t)r * hidden;
    float x[CH][4], d[CH][4];
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * 32 + lane) * 4;
        if (i < hidden) Vec<float, 4>::load(residual + row + i, x[c]);
    }
    if (delta) {
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            const int i = (c * 32 + lane) * 4;
            if (i < hidden) Vec<TD, 4>::load(delta + row + i, d[c]);
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * 32 + lane) * 4;
        if (i < hidden) {
            if (delta) {
#pragma unroll
                for (int k = 0; k < 4; ++k) x[c][k] += d[c][k];
                Vec<float, 4>::store(residual + row + i, x[c]);
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) ss += x[c][k] * x[c][k];
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!out) return;
    const float factor = rsqrtf(ss / (float)hidden + eps);
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * 32 + lane) * 4;
        if (i < hidden) {
            float y[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) y[k] = x[c][k] * factor * s_gain[i + k];
            Vec<TO, 4>::store(out + row + i, y);
        }
    }
}

// ---- gather of wanted rows ------------------------------------------------------------------------
// out[s, :] = residual[idx[s], :] (+ scale * (delta[idx[s], :] (+ delta2[idx[s], :]))) in 32 bits.
template <typename TD>
__global__ void gather_rows_kernel(const float* __restrict__ residual, const TD* __restrict__ delta,
                                   const TD* __restrict__ delta2, float scale, const int* __restrict__ idx,
                                   float* __restrict__ out, int hidden, int num_rows) {
    const int s = blockIdx.x;
    int r = idx[s];
    if (r < 0 || r >= num_rows) r = 0;
    const size_t src = (size_t)r * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float v = residual[src + i];
        if (delta) {
            float d = to_f32(delta[src + i]);
            if (delta2) d += to_f32(delta2[src + i]);
            v = fmaf(scale, d, v);
        }
        out[(size_t)s * hidden + i] = v;
    }
}

// ---- SiLU-gated product ---------------------------------------------------------------------------
// act[t, j] = silu(gate_up[t, j]) * gate_up[t, I + j], silu(g) = g / (1 + exp(-g)), in 32 bits with the
// exact exponential.
template <typename T, int V>
__global__ void silu_mul_kernel(const T* __restrict__ gate_up, T* __restrict__ act, int inter, int rows, int gelu) {
    const int per_row = inter / V;
    const size_t total = (size_t)rows * per_row;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total;
         e += (size_t)gridDim.x * blockDim.x) {
        const size_t t = e / per_row;
        const int j = (int)(e % per_row) * V;
        float g[V], u[V];
        Vec<T, V>::load(gate_up + t * 2 * inter + j, g);
        Vec<T, V>::load(gate_up + t * 2 * inter + inter + j, u);
#pragma unroll
        for (int k = 0; k < V; ++k)
            g[k] = (gelu ? 0.5f * g[k] * (1.f + tanhf(0.7978845608028654f * (g[k] + 0.044715f * g[k] * g[k] * g[k])))
                         : g[k] / (1.f + expf(-g[k]))) * u[k];
        Vec<T, V>::store(act + t * inter + j, g);
    }
}

// ---- squared ReLU ------------------------------------------------------------------------------------
// out = max(x, 0)^2, taken in 32 bits and rounded once.
template <typename T>
__global__ void relu_squared_kernel(const T* __restrict__ x, T* __restrict__ out, size_t total) {
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
        const float v = fmaxf(to_f32(x[e]), 0.f);
        out[e] = from_f32<T>(v * v);
    }
}

// out = x + bias, or max(x + bias, 0)^2 (`squared_relu`), for rows of `cols` values; 32-bit with one rounding; out may be x.
template <typename T, int V>
__global__ void bias_rows_kernel(const T* x, const float* __restrict__ bias, T* out, int cols, size_t total, int squared_relu) {
    griddep_launch();
    griddep_wait();
    for (size_t e = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V; e < total; e += (size_t)gridDim.x * blockDim.x * V) {
        const int j = (int)(e % cols);
        float v[V];
        Vec<T, V>::load(x + e, v);
#pragma unroll
        for (int k = 0; k < V; ++k) {
            v[k] += bias[j + k];
            if (squared_relu) {
                v[k] = fmaxf(v[k], 0.f);
                v[k] *= v[k];
            }
        }
        Vec<T, V>::store(out + e, v);
    }
}

// out = scale_a * a + scale_b * b, 32-bit with one rounding.
template <typename T, int V>
__global__ void pair_sum_kernel(const T* __restrict__ a, const T* __restrict__ b, float scale_a, float scale_b, T* __restrict__ out, size_t total) {
    griddep_launch();
    griddep_wait();
    for (size_t e = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V; e < total; e += (size_t)gridDim.x * blockDim.x * V) {
        float x[V], y[V];
        Vec<T, V>::load(a + e, x);
        Vec<T, V>::load(b + e, y);
#pragma unroll
        for (int k = 0; k < V; ++k) x[k] = scale_a * x[k] + scale_b * y[k];
        Vec<T, V>::store(out + e, x);
    }
}

// ---- sigmoid gate -------------------------------------------------------------------------------------
// out[t, j] = x[t, j] * sigmoid(gate[t, j]) with the exact exponential; the rows of x and of gate may lie inside wider
// rows (their strides are given), out is dense.
template <typename T>
__global__ void sigmoid_gate_kernel(const T* __restrict__ x, int x_stride, const T* __restrict__ gate, int gate_stride,
                                    T* __restrict__ out, int cols, int rows) {
    const size_t total = (size_t)rows * cols;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
        const size_t t = e / cols;
        const int j = (int)(e % cols);
        const float g = to_f32(gate[t * gate_stride + j]);
        out[e] = from_f32<T>(to_f32(x[t * x_stride + j]) / (1.f + expf(-g)));
    }
}

}  // namespace cib

using namespace cib;

static inline int flat_blocks(size_t total) {
    size_t b = (total + 255) / 256;
    return (int)(b > 148 * 16 ? 148 * 16 : (b ? b : 1));
}

extern "C" int cib_relu_squared(const void* x, void* out, int dtype, long long total, cudaStream_t stream) {
    CIB_REQUIRE(total >= 0, "relu_squared: bad size");
    if (total == 0) return 0;
    if (dtype == kF32) relu_squared_kernel<float><<<flat_blocks(total), 256, 0, stream>>>((const float*)x, (float*)out, (size_t)total);
    else if (dtype == kBF16) relu_squared_kernel<__nv_bfloat16><<<flat_blocks(total), 256, 0, stream>>>((const __nv_bfloat16*)x, (__nv_bfloat16*)out, (size_t)total);
    else CIB_REQUIRE(false, "relu_squared: unsupported dtype %d", dtype);
    CIB_LAUNCH_CHECK("relu_squared");
    return 0;
}

// x, out [rows][cols] (out may be x); bias float32 [cols].
extern "C" int cib_bias_rows(const void* x, const float* bias, void* out, int dtype, int rows, int cols, int squared_relu, cudaStream_t stream) {
    CIB_REQUIRE(rows >= 0 && cols > 0 && bias, "bias_rows: bad arguments");
    if (rows == 0) return 0;
    const size_t total = (size_t)rows * cols;
    const bool v4 = cols % 4 == 0, pdl = prompt_pdl();
#define CIB_BIAS(T, V) launch_pdl(bias_rows_kernel<T, V>, dim3(flat_blocks(total / V)), dim3(256), 0, stream, pdl, (const T*)x, bias, (T*)out, cols, total, squared_relu)
    if (dtype == kF32) { if (v4) CIB_BIAS(float, 4); else CIB_BIAS(float, 1); }
    else if (dtype == kBF16) { if (v4) CIB_BIAS(__nv_bfloat16, 4); else CIB_BIAS(__nv_bfloat16, 1); }
    else CIB_REQUIRE(false, "bias_rows: bad dtype %d", dtype);
#undef CIB_BIAS
    CIB_LAUNCH_CHECK("bias_rows");
    return 0;
}

extern "C" int cib_pair_sum(const void* a, const void* b, float scale_a, float scale_b, void* out, int dtype, long long total,
                            cudaStream_t stream) {
    CIB_REQUIRE(total >= 0, "pair_sum: bad size");
    if (total == 0) return 0;
    const bool v4 = total % 4 == 0, pdl = prompt_pdl();
#define CIB_PAIR_SUM(T, V) launch_pdl(pair_sum_kernel<T, V>, dim3(flat_blocks((size_t)total / V)), dim3(256), 0, stream, pdl, (const T*)a, (const T*)b, scale_a, scale_b, (T*)out, (size_t)total)
    if (dtype == kF32) { if (v4) CIB_PAIR_SUM(float, 4); else CIB_PAIR_SUM(float, 1); }
    else if (dtype == kBF16) { if (v4) CIB_PAIR_SUM(__nv_bfloat16, 4); else CIB_PAIR_SUM(__nv_bfloat16, 1); }
    else CIB_REQUIRE(false, "pair_sum: bad dtype %d", dtype);
#undef CIB_PAIR_SUM
    CIB_LAUNCH_CHECK("pair_sum");
    return 0;
}

extern "C" int cib_sigmoid_gate(const void* x, int x_stride, const void* gate, int gate_stride, void* out, int dtype,
                                int rows, int cols, cudaStream_t stream) {
    CIB_REQUIRE(rows >= 0 && cols > 0 && x_stride >= cols && gate_stride >= cols, "sigmoid_gate: bad sizes rows=%d cols=%d", rows, cols);
    if (rows == 0) return 0;
    const size_t total = (size_t)rows * cols;
    if (dtype == kF32) sigmoid_gate_kernel<float><<<flat_blocks(total), 256, 0, stream>>>((const float*)x, x_stride, (const float*)gate, gate_stride, (float*)out, cols, rows);
    else if (dtype == kBF16) sigmoid_gate_kernel<__nv_bfloat16><<<flat_blocks(total), 256, 0, stream>>>((const __nv_bfloat16*)x, x_stride, (const __nv_bfloat16*)gate, gate_stride, (__nv_bfloat16*)out, cols, rows);
    else CIB_REQUIRE(false, "sigmoid_gate: unsupported dtype %d", dtype);
    CIB_LAUNCH_CHECK("sigmoid_gate");
    return 0;
}

static inline int norm_threads(int hidden, int vec) {
    int per = (hidden + vec - 1) / vec;
    int t = 32;
    while (t < per && t < 1024) t <<= 1;
    return t;
}

extern "C" int cib_embedding_gather(const int* ids, const void* table, int table_dtype, float* out,
                                    int num_tokens, int hidden, int vocab, int* bad_flag, float scale, int copies,
                                    cudaStream_t stream) {
    CIB_REQUIRE(num_tokens >= 0 && hidden > 0 && vocab > 0 && copies >= 1, "embedding_gather: bad sizes T=%d H=%d V=%d",
                num_tokens, hidden, vocab);
    if (num_tokens == 0) return 0;
    const bool v4 = hidden % 4 == 0;
    const int threads = norm_threads(hidden, v4 ? 4 : 1) > 256 ? 256 : norm_threads(hidden, v4 ? 4 : 1);
    if (table_dtype == kF32) {
        if (v4) embedding_gather_kernel<float, 4><<<num_tokens, threads, 0, stream>>>(ids, (const float*)table, out, hidden, vocab, bad_flag, scale, copies);
        else embedding_gather_kernel<float, 1><<<num_tokens, threads, 0, stream>>>(ids, (const float*)table, out, hidden, vocab, bad_flag, scale, copies);
    } else if (table_dtype == kBF16) {
        if (v4) embedding_gather_kernel<__nv_bfloat16, 4><<<num_tokens, threads, 0, stream>>>(ids, (const __nv_bfloat16*)table, out, hidden, vocab, bad_flag, scale, copies);
        else embedding_gather_kernel<__nv_bfloat16, 1><<<num_tokens, threads, 0, stream>>>(ids, (const __nv_bfloat16*)table, out, hidden, vocab, bad_flag, scale, copies);
    } else {
        CIB_REQUIRE(false, "embedding_gather: unsupported table dtype %d", table_dtype);
    }
    CIB_LAUNCH_CHECK("embedding_gather");
    return 0;
}

template <typename TD, typename TO>
static void launch_add_rmsnorm(float* residual, const void* delta, AnyVec w, float eps, void* out, int rows,
                               int hidden, cudaStream_t stream) {
    // from 256 rows on and up to 2048 values a row: a warp per row
    if (hidden % 4 == 0 && rows >= 256 && hidden <= 2048) {
        const int ch = (hidden + 127) / 128;
        const dim3 grid((rows + 7) / 8);
        const bool pdl = prompt_pdl();
        if (ch <= 4) launch_pdl(add_rmsnorm_rows_kernel<TD, TO, 4>, dim3(grid), dim3(256), 0, stream, pdl, residual, (const TD*)delta, w, eps, (TO*)out, hidden, rows);
        else if (ch <= 8) launch_pdl(add_rmsnorm_rows_kernel<TD, TO, 8>, dim3(grid), dim3(256), 0, stream, pdl, residual, (const TD*)delta, w, eps, (TO*)out, hidden, rows);
        else launch_pdl(add_rmsnorm_rows_kernel<TD, TO, 16>, dim3(grid), dim3(256), 0, stream, pdl, residual, (const TD*)delta, w, eps, (TO*)out, hidden, rows);
    } else if (hidden % 4 == 0) {
        add_rmsnorm_kernel<TD, TO, 4><<<rows, norm_threads(hidden, 4), 0, stream>>>(residual, (const TD*)delta, w, eps, (TO*)out, hidden);
    } else {
        add_rmsnorm_kernel<TD, TO, 1><<<rows, norm_threads(hidden, 1), 0, stream>>>(residual, (const TD*)delta, w, eps, (TO*)out, hidden);
    }
}

// delta may be null (plain norm of the residual rows); out may be null (add only).
extern "C" int cib_add_rmsnorm(float* residual, const void* delta, int delta_dtype, const void* weight,
                               int weight_dtype, float eps, void* out, int out_dtype, int rows, int hidden,
                               cudaStream_t stream) {
    CIB_REQUIRE(rows >= 0 && hidden > 0, "add_rmsnorm: bad sizes rows=%d hidden=%d", rows, hidden);
    CIB_REQUIRE(out == nullptr || weight != nullptr, "add_rmsnorm: a norm needs its weight");
    if (rows == 0) return 0;
    AnyVec w{weight, weight_dtype == kBF16};
    const int dd = delta ? delta_dtype : kF32;
    if (dd == kF32 && out_dtype == kF32) launch_add_rmsnorm<float, float>(residual, delta, w, eps, out, rows, hidden, stream);
    else if (dd == kF32 && out_dtype == kBF16) launch_add_rmsnorm<float, __nv_bfloat16>(residual, delta, w, eps, out, rows, hidden, stream);
    else if (dd == kBF16 && out_dtype == kF32) launch_add_rmsnorm<__nv_bfloat16, float>(residual, delta, w, eps, out, rows, hidden, stream);
    else if (dd == kBF16 && out_dtype == kBF16) launch_add_rmsnorm<__nv_bfloat16, __nv_bfloat16>(residual, delta, w, eps, out, rows, hidden, stream);
    else CIB_REQUIRE(false, "add_rmsnorm: unsupported dtypes delta=%d out=%d", delta_dtype, out_dtype);
    CIB_LAUNCH_CHECK("add_rmsnorm");
    return 0;
}

extern "C" int cib_gather_rows(const float* residual, const void* delta, const void* delta2, int delta_dtype, float scale,
                               const int* idx, float* out, int num_out, int hidden, int num_rows, cudaStream_t stream) {
    CIB_REQUIRE(num_out >= 0 && hidden > 0, "gather_rows: bad sizes");
    CIB_REQUIRE(delta || !delta2, "gather_rows: a second delta needs a first one");
    if (num_out == 0) return 0;
    const int threads = hidden >= 256 ? 256 : 64;
    if (!delta || delta_dtype == kF32) gather_rows_kernel<float><<<num_out, threads, 0, stream>>>(residual, (const float*)delta, (const float*)delta2, scale, idx, out, hidden, num_rows);
    else if (delta_dtype == kBF16) gather_rows_kernel<__nv_bfloat16><<<num_out, threads, 0, stream>>>(residual, (const __nv_bfloat16*)delta, (const __nv_bfloat16*)delta2, scale, idx, out, hidden, num_rows);
    else CIB_REQUIRE(false, "gather_rows: unsupported delta dtype %d", delta_dtype);
    CIB_LAUNCH_CHECK("gather_rows");
    return 0;
}

// gelu != 0: the gate goes through the tanh form of GELU instead of SiLU (exact tangent).
extern "C" int cib_silu_mul(const void* gate_up, void* act, int dtype, int rows, int inter, int gelu, cudaStream_t stream) {
    CIB_REQUIRE(rows >= 0 && inter > 0, "silu_mul: bad sizes rows=%d I=%d", rows, inter);
    if (rows == 0) return 0;
    const bool v4 = inter % 4 == 0;
    const size_t total = (size_t)rows * (inter / (v4 ? 4 : 1));
    int blocks = (int)((total + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == kF32) {
        if (v4) silu_mul_kernel<float, 4><<<blocks, 256, 0, stream>>>((const float*)gate_up, (float*)act, inter, rows, gelu);
        else silu_mul_kernel<float, 1><<<blocks, 256, 0, stream>>>((const float*)gate_up, (float*)act, inter, rows, gelu);
    } else if (dtype == kBF16) {
        if (v4) silu_mul_kernel<__nv_bfloat16, 4><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)gate_up, (__nv_bfloat16*)act, inter, rows, gelu);
        else silu_mul_kernel<__nv_bfloat16, 1><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)gate_up, (__nv_bfloat16*)act, inter, rows, gelu);
    } else {
        CIB_REQUIRE(false, "silu_mul: unsupported dtype %d", dtype);
    }
    CIB_LAUNCH_CHECK("silu_mul");
    return 0;
}

// ---- RMS norms on both sides of the residual sum ---------------------------------------------------------------------
// One pass over a 32-bit residual row x with an outstanding delta y (either may be absent):
//   x += post ? y * rsqrt(mean(y^2) + post_eps) * post_gain : y          (a sub-layer's output, normed before it is added)
//   raw  = x rounded to the rows' type                                   (for a part that reads the stream itself)
//   out  = x * rsqrt(mean(x^2) + eps) * gain                             (the next sub-layer's input)
// Statistics 32-bit; a block per row, the row staged in shared memory.
namespace cib {

template <typename TD, typename TO>
__global__ void __launch_bounds__(256)
rms_stream_kernel(float* __restrict__ residual, const TD* __restrict__ delta, AnyVec post_gain, int has_post, float post_eps,
                  AnyVec gain, float eps, TO* __restrict__ out, TO* __restrict__ raw, int hidden) {
    extern __shared__ float row_s[];
    __shared__ float scratch[33];
    const size_t row = (size_t)blockIdx.x * hidden;
    float factor = 1.f;
    if (delta && has_post) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
            const float y = to_f32(delta[row + i]);
            ss = fmaf(y, y, ss);
        }
        ss = block_sum(ss, scratch);
        factor = 1.f / sqrtf(ss / (float)hidden + post_eps);
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float x = residual[row + i];
        if (delta) {
            const float y = to_f32(delta[row + i]);
            x += has_post ? y * factor * post_gain[i] : y;
            residual[row + i] = x;
        }
        row_s[i] = x;
        ss = fmaf(x, x, ss);
        if (raw) raw[row + i] = from_f32<TO>(x);
    }
    if (!out) return;
    ss = block_sum(ss, scratch);
    const float f2 = 1.f / sqrtf(ss / (float)hidden + eps);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) out[row + i] = from_f32<TO>(row_s[i] * f2 * gain[i]);
}

// Rows of a multiple of four values: four a lane and load, the row (CH * 4 values a thread) in registers, every load issued
// before the first use; the gains come after the reductions.
template <typename TD, typename TO, int CH>
__global__ void __launch_bounds__(256)
rms_stream_vec_kernel(float* __restrict__ residual, const TD* __restrict__ delta, AnyVec post_gain, int has_post, float post_eps,
                      AnyVec gain, float eps, TO* __restrict__ out, TO* __restrict__ raw, int hidden) {
    __shared__ float scratch[33];
    griddep_launch();
    griddep_wait();
    const size_t row = (size_t)blockIdx.x * hidden;
    float x[CH][4], y[CH][4];
    auto at = [&](int c) { return (c * (int)blockDim.x + (int)threadIdx.x) * 4; };
#pragma unroll
    for (int c = 0; c < CH; ++c)
        if (at(c) < hidden) Vec<float, 4>::load(residual + row + at(c), x[c]);
    if (delta) {
#pragma unroll
        for (int c = 0; c < CH; ++c)
            if (at(c) < hidden) Vec<TD, 4>::load(delta + row + at(c), y[c]);
        float factor = 1.f;
        if (has_post) {
            float ss = 0.f;
#pragma unroll
            for (int c = 0; c < CH; ++c)
                if (at(c) < hidden) {
#pragma unroll
                    for (int k = 0; k < 4; ++k) ss = fmaf(y[c][k], y[c][k], ss);
                }
            ss = block_sum(ss, scratch);
            factor = 1.f / sqrtf(ss / (float)hidden + post_eps);
        }
#pragma unroll
        for (int c = 0; c < CH; ++c)
            if (at(c) < hidden) {
#pragma unroll
                for (int k = 0; k < 4; ++k) x[c][k] += has_post ? y[c][k] * factor * post_gain[at(c) + k] : y[c][k];
                Vec<float, 4>::store(residual + row + at(c), x[c]);
            }
    }
    if (raw) {
#pragma unroll
        for (int c = 0; c < CH; ++c)
            if (at(c) < hidden) Vec<TO, 4>::store(raw + row + at(c), x[c]);
    }
    if (!out) return;
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c)
        if (at(c) < hidden) {
#pragma unroll
            for (int k = 0; k < 4; ++k) ss = fmaf(x[c][k], x[c][k], ss);
        }
    ss = block_sum(ss, scratch);
    const float f2 = 1.f / sqrtf(ss / (float)hidden + eps);
#pragma unroll
    for (int c = 0; c < CH; ++c)
        if (at(c) < hidden) {
#pragma unroll
            for (int k = 0; k < 4; ++k) y[c][k] = x[c][k] * f2 * gain[at(c) + k];
            Vec<TO, 4>::store(out + row + at(c), y[c]);
        }
}

// out[t, j] = gelu_tanh(x[t, j]) (* table[ids[t], j] when a table is given);
// gelu_tanh(z) = 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))), 32-bit with the exact tangent.
template <typename T>
__global__ void gelu_tanh_kernel(const T* __restrict__ x, const T* __restrict__ table, int table_stride,
                                 const int* __restrict__ ids, int vocab, T* __restrict__ out, int cols, long long total) {
    for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
        const float z = to_f32(x[e]);
        float y = 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
        if (table) {
            const long long t = e / cols;
            const int id = ids[t];
            y = (id >= 0 && id < vocab) ? y * to_f32(table[(size_t)id * table_stride + (e - t * cols)]) : 0.f;
        }
        out[e] = from_f32<T>(y);
    }
}

}  // namespace cib

extern "C" int cib_rms_stream(float* residual, const void* delta, int delta_dtype, const void* post_gain, int post_dtype,
                              float post_eps, const void* gain, int gain_dtype, float eps, void* out, void* raw,
                              int out_dtype, int rows, int hidden, cudaStream_t stream) {
    using namespace cib;
    CIB_REQUIRE(rows >= 0 && hidden > 0 && hidden <= 12 * 1024, "rms_stream: bad sizes (%d x %d)", rows, hidden);
    CIB_REQUIRE(!post_gain || delta, "rms_stream: an output norm needs rows to norm");
    CIB_REQUIRE(!out || gain, "rms_stream: out needs the norm's gain");
    if (rows == 0) return 0;
    AnyVec pg{post_gain, post_dtype == kBF16}, g{gain, gain_dtype == kBF16};
    const size_t smem = (size_t)hidden * sizeof(float);
    const int has_post = post_gain != nullptr;
    // up to 1 024 values a row: as many threads as it has fours; beyond, 256 threads with up to eight fours each
    const bool vec = hidden % 4 == 0 && hidden <= 8192, pdl = prompt_pdl();
    const int threads = hidden >= 1024 ? 256 : std::max(32, (hidden / 4 + 31) / 32 * 32);
#define CIB_RMS_VEC(TD, TO, CH)                                                                                                  \
    launch_pdl(rms_stream_vec_kernel<TD, TO, CH>, dim3(rows), dim3(threads), 0, stream, pdl, residual, (const TD*)delta, pg, has_post,  \
               post_eps, g, eps, (TO*)out, (TO*)raw, hidden)
#define CIB_RMS_STREAM(TD, TO)                                                                                                   \
    do {                                                                                                                         \
        if (vec && hidden <= 1024) CIB_RMS_VEC(TD, TO, 1);                                                                       \
        else if (vec && hidden <= 2048) CIB_RMS_VEC(TD, TO, 2);                                                                  \
        else if (vec && hidden <= 4096) CIB_RMS_VEC(TD, TO, 4);                                                                  \
        else if (vec) CIB_RMS_VEC(TD, TO, 8);                                                                                    \
        else rms_stream_kernel<TD, TO><<<rows, 256, smem, stream>>>(residual, (const TD*)delta, pg, has_post, post_eps, g, eps, (TO*)out, (TO*)raw, hidden); \
    } while (0)
    const bool d16 = delta && delta_dtype == kBF16, o16 = out_dtype == kBF16;
    if (d16 && o16) CIB_RMS_STREAM(__nv_bfloat16, __nv_bfloat16);
    else if (d16) CIB_RMS_STREAM(__nv_bfloat16, float);
    else if (o16) CIB_RMS_STREAM(float, __nv_bfloat16);
    else CIB_RMS_STREAM(float, float);
#undef CIB_RMS_STREAM
#undef CIB_RMS_VEC
    CIB_LAUNCH_CHECK("rms_stream");
    return 0;
}

extern "C" int cib_gelu_tanh(const void* x, const void* table, int table_stride, const int* ids, int vocab, void* out, int dtype,
                             int rows, int cols, cudaStream_t stream) {
    using namespace cib;
    CIB_REQUIRE(rows >= 0 && cols > 0 && (!table || ids), "gelu_tanh: bad arguments");
    const long long total = (long long)rows * cols;
    if (total == 0) return 0;
    const int blocks = (int)std::min<long long>((total + 255) / 256, 148 * 16);
    if (dtype == kF32)
        gelu_tanh_kernel<float><<<blocks, 256, 0, stream>>>((const float*)x, (const float*)table, table_stride, ids, vocab, (float*)out, cols, total);
    else if (dtype == kBF16)
        gelu_tanh_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)x, (const __nv_bfloat16*)table, table_stride, ids, vocab, (__nv_bfloat16*)out, cols, total);
    else
        CIB_REQUIRE(false, "gelu_tanh: bad dtype %d", dtype);
    CIB_LAUNCH_CHECK("gelu_tanh");
    return 0;
}

// ---- a scaled residual sum of two deltas, and an RMS norm in groups ------------------------------------------------------
// One pass over the 32-bit residual rows x:
//   x   += scale * (delta + delta2)                         (either delta may be absent)
//   out  = part / sqrt(mean(part^2) + eps) * gain           for each of `groups` equal consecutive parts of the row
// The parts of a row are independent, so the kernels walk rows * groups parts of hidden / groups values whose gains start
// at (part % groups) * width.  Statistics and sum 32-bit, one rounding at the end.
namespace cib {

// Few parts: a block per part.
template <typename TD, typename TO, int V>
__global__ void group_rms_kernel(float* __restrict__ residual, const TD* __restrict__ delta, const TD* __restrict__ delta2,
                                 float scale, AnyVec gain, float eps, TO* __restrict__ out, int groups, int width) {
    __shared__ float scratch[33];
    griddep_launch();
    griddep_wait();
    const size_t at = (size_t)blockIdx.x * width;
    const int g0 = (int)(blockIdx.x % groups) * width;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float x[V];
        Vec<float, V>::load(residual + at + i, x);
        if (delta) {
            float d[V];
            Vec<TD, V>::load(delta + at + i, d);
            if (delta2) {
                float e[V];
                Vec<TD, V>::load(delta2 + at + i, e);
#pragma unroll
                for (int k = 0; k < V; ++k) d[k] += e[k];
            }
#pragma unroll
            for (int k = 0; k < V; ++k) x[k] = fmaf(scale, d[k], x[k]);
            Vec<float, V>::store(residual + at + i, x);
        }
#pragma unroll
        for (int k = 0; k < V; ++k) ss += x[k] * x[k];
    }
    if (!out) return;
    ss = block_sum(ss, scratch);
    const float factor = 1.f / sqrtf(ss / (float)width + eps);
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float x[V];
        Vec<float, V>::load(residual + at + i, x);          // this thread wrote exactly these elements above
#pragma unroll
        for (int k = 0; k < V; ++k) x[k] = x[k] * factor * gain[g0 + i + k];
        Vec<TO, V>::store(out + at + i, x);
    }
}

// Many parts of up to CH * 128 values: a warp per part, the part in registers, every load issued before the first use.
template <typename TD, typename TO, int CH>
__global__ void __launch_bounds__(256)
group_rms_rows_kernel(float* __restrict__ residual, const TD* __restrict__ delta, const TD* __restrict__ delta2, float scale,
                      AnyVec gain, float eps, TO* __restrict__ out, int groups, int width, long long parts) {
    griddep_launch();
    griddep_wait();
    const int lane = threadIdx.x & 31;
    const long long part = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (part >= parts) return;
    const size_t at = (size_t)part * width;
    const int g0 = (int)(part % groups) * width;
    float x[CH][4], d[CH][4];
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * 32 + lane) * 4;
        if (i < width) Vec<float, 4>::load(residual + at + i, x[c]);
    }
    if (delta) {
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            const int i = (c * 32 + lane) * 4;
            if (i < width) Vec<TD, 4>::load(delta + at + i, d[c]);
        }
        if (delta2) {
#pragma unroll
            for (int c = 0; c < CH; ++c) {
                const int i = (c * 32 + lane) * 4;
                if (i < width) {
                    float e[4];
                    Vec<TD, 4>::load(delta2 + at + i, e);
#pragma unroll
                    for (int k = 0; k < 4; ++k) d[c][k] += e[k];
                }
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * 32 + lane) * 4;
        if (i < width) {
            if (delta) {
#pragma unroll
                for (int k = 0; k < 4; ++k) x[c][k] = fmaf(scale, d[c][k], x[c][k]);
                Vec<float, 4>::store(residual + at + i, x[c]);
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) ss += x[c][k] * x[c][k];
        }
    }
    if (!out) return;
    ss = warp_sum(ss);
    const float factor = 1.f / sqrtf(ss / (float)width + eps);
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * 32 + lane) * 4;
        if (i < width) {
            float y[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) y[k] = x[c][k] * factor * gain[g0 + i + k];
            Vec<TO, 4>::store(out + at + i, y);
        }
    }
}

template <typename TD, typename TO>
static void launch_group_rms(float* residual, const void* delta, const void* delta2, float scale, AnyVec gain, float eps, void* out,
                             int rows, int hidden, int groups, cudaStream_t stream) {
    const int width = hidden / groups;
    const long long parts = (long long)rows * groups;
    const bool pdl = prompt_pdl();
    const TD *d1 = (const TD*)delta, *d2 = (const TD*)delta2;
    if (width % 4 == 0 && parts >= 256 && width <= 2048) {
        const int ch = (width + 127) / 128;
        const dim3 grid((unsigned)((parts + 7) / 8));
        if (ch <= 4) launch_pdl(group_rms_rows_kernel<TD, TO, 4>, grid, dim3(256), 0, stream, pdl, residual, d1, d2, scale, gain, eps, (TO*)out, groups, width, parts);
        else if (ch <= 8) launch_pdl(group_rms_rows_kernel<TD, TO, 8>, grid, dim3(256), 0, stream, pdl, residual, d1, d2, scale, gain, eps, (TO*)out, groups, width, parts);
        else launch_pdl(group_rms_rows_kernel<TD, TO, 16>, grid, dim3(256), 0, stream, pdl, residual, d1, d2, scale, gain, eps, (TO*)out, groups, width, parts);
    } else if (width % 4 == 0) {
        launch_pdl(group_rms_kernel<TD, TO, 4>, dim3((unsigned)parts), dim3(norm_threads(width, 4)), 0, stream, pdl, residual, d1, d2, scale, gain, eps, (TO*)out, groups, width);
    } else {
        launch_pdl(group_rms_kernel<TD, TO, 1>, dim3((unsigned)parts), dim3(norm_threads(width, 1)), 0, stream, pdl, residual, d1, d2, scale, gain, eps, (TO*)out, groups, width);
    }
}

// ---- half the sum of two rows, each RMS-normed over the whole row ------------------------------------------------------------
// out[t] = 1/2 (a / sqrt(mean(a^2) + eps) * gain_a + b / sqrt(mean(b^2) + eps) * gain_b): a block per row.
template <typename T, int V>
__global__ void __launch_bounds__(256)
pair_rms_mean_kernel(const T* __restrict__ a, const T* __restrict__ b, AnyVec gain_a, AnyVec gain_b, float eps,
                     T* __restrict__ out, int hidden) {
    __shared__ float scratch[33];
    griddep_launch();
    griddep_wait();
    const size_t at = (size_t)blockIdx.x * hidden;
    float sa = 0.f, sb = 0.f;
    for (int i = threadIdx.x * V; i < hidden; i += blockDim.x * V) {
        float x[V], y[V];
        Vec<T, V>::load(a + at + i, x);
        Vec<T, V>::load(b + at + i, y);
#pragma unroll
        for (int k = 0; k < V; ++k) {
            sa = fmaf(x[k], x[k], sa);
            sb = fmaf(y[k], y[k], sb);
        }
    }
    sa = block_sum(sa, scratch);
    sb = block_sum(sb, scratch);
    const float fa = 0.5f / sqrtf(sa / (float)hidden + eps), fb = 0.5f / sqrtf(sb / (float)hidden + eps);
    for (int i = threadIdx.x * V; i < hidden; i += blockDim.x * V) {
        float x[V], y[V];
        Vec<T, V>::load(a + at + i, x);
        Vec<T, V>::load(b + at + i, y);
#pragma unroll
        for (int k = 0; k < V; ++k) x[k] = x[k] * fa * gain_a[i + k] + y[k] * fb * gain_b[i + k];
        Vec<T, V>::store(out + at + i, x);
    }
}

// out = tanh(x), 32-bit in with the exact tangent, one rounding at the end.
template <typename T>
__global__ void tanh_rows_kernel(const float* __restrict__ x, int x_stride, T* __restrict__ out, int cols, long long total) {
    for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
        const long long t = e / cols;
        out[e] = from_f32<T>(tanhf(x[t * x_stride + (e - t * cols)]));
    }
}

}  // namespace cib

// delta, delta2 (of one type) may be null; out may be null (the sum alone).
extern "C" int cib_group_rms(float* residual, const void* delta, const void* delta2, int delta_dtype, float scale, const void* gain,
                             int gain_dtype, float eps, int groups, void* out, int out_dtype, int rows, int hidden,
                             cudaStream_t stream) {
    CIB_REQUIRE(rows >= 0 && hidden > 0 && groups > 0 && hidden % groups == 0, "group_rms: bad sizes (%d x %d in %d groups)", rows, hidden, groups);
    CIB_REQUIRE(delta || !delta2, "group_rms: a second delta needs a first one");
    CIB_REQUIRE(!out || gain, "group_rms: a norm needs its gain");
    CIB_REQUIRE((long long)rows * groups < (1ll << 31), "group_rms: too many rows");
    if (rows == 0 || (!delta && !out)) return 0;
    AnyVec g{gain, gain_dtype == kBF16};
    const bool d16 = delta && delta_dtype == kBF16, o16 = out_dtype == kBF16;
    if (d16 && o16) launch_group_rms<__nv_bfloat16, __nv_bfloat16>(residual, delta, delta2, scale, g, eps, out, rows, hidden, groups, stream);
    else if (d16) launch_group_rms<__nv_bfloat16, float>(residual, delta, delta2, scale, g, eps, out, rows, hidden, groups, stream);
    else if (o16) launch_group_rms<float, __nv_bfloat16>(residual, delta, delta2, scale, g, eps, out, rows, hidden, groups, stream);
    else launch_group_rms<float, float>(residual, delta, delta2, scale, g, eps, out, rows, hidden, groups, stream);
    CIB_LAUNCH_CHECK("group_rms");
    return 0;
}

extern "C" int cib_pair_rms_mean(const void* a, const void* b, int dtype, const void* gain_a, const void* gain_b, int gain_dtype,
                                 float eps, void* out, int rows, int hidden, cudaStream_t stream) {
    CIB_REQUIRE(rows >= 0 && hidden > 0, "pair_rms_mean: bad sizes");
    if (rows == 0) return 0;
    AnyVec ga{gain_a, gain_dtype == kBF16}, gb{gain_b, gain_dtype == kBF16};
    const bool pdl = prompt_pdl();
#define CIB_PAIR(T, V)                                                                                                         \
    launch_pdl(pair_rms_mean_kernel<T, V>, dim3(rows), dim3(std::min(256, norm_threads(hidden, V))), 0, stream, pdl, (const T*)a,     \
               (const T*)b, ga, gb, eps, (T*)out, hidden)
    if (dtype == kF32) {
        if (hidden % 4 == 0) CIB_PAIR(float, 4);
        else CIB_PAIR(float, 1);
    } else if (dtype == kBF16) {
        if (hidden % 4 == 0) CIB_PAIR(__nv_bfloat16, 4);
        else CIB_PAIR(__nv_bfloat16, 1);
    } else {
        CIB_REQUIRE(false, "pair_rms_mean: bad dtype %d", dtype);
    }
#undef CIB_PAIR
    CIB_LAUNCH_CHECK("pair_rms_mean");
    return 0;
}

extern "C" int cib_tanh_rows(const float* x, int x_stride, void* out, int out_dtype, int rows, int cols, cudaStream_t stream) {
    CIB_REQUIRE(rows >= 0 && cols > 0 && x_stride >= cols, "tanh_rows: bad sizes");
    const long long total = (long long)rows * cols;
    if (total == 0) return 0;
    const int blocks = (int)std::min<long long>((total + 255) / 256, 148 * 16);
    if (out_dtype == kF32) tanh_rows_kernel<float><<<blocks, 256, 0, stream>>>(x, x_stride, (float*)out, cols, total);
    else if (out_dtype == kBF16) tanh_rows_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>(x, x_stride, (__nv_bfloat16*)out, cols, total);
    else CIB_REQUIRE(false, "tanh_rows: bad dtype %d", out_dtype);
    CIB_LAUNCH_CHECK("tanh_rows");
    return 0;
}
