// What the scans over a matrix state share (recurrent.cu, recurrent_channel.cu): scalar functions, how a column of the
// state is laid over lanes, and the layout of the staging rows.
#pragma once

#include "common.cuh"

namespace cib {

__device__ __forceinline__ float sigmoidf_(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplusf_(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float logsigmoidf_(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

constexpr int kScanWarps = 4;
constexpr int kScanChunk = 16;          // tokens staged in shared memory at a time

// index of key element i in the staging rows: four floats of padding after every 32, so that the lanes of a column
// (which read elements 32 apart, four at a time) hit different banks
__device__ __forceinline__ int pad32(int i) { return i + 4 * (i >> 5); }
template <int DP> constexpr int padded_len() { return DP + 4 * (DP / 32); }

template <int SPLIT>
__device__ __forceinline__ float split_sum(float v) {
#pragma unroll
    for (int o = SPLIT / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

}  // namespace cib

// calls CALL with DP, the key size rounded up to a compiled one
#define CIB_SCAN_DISPATCH(d, CALL)                         \
    do {                                                   \
        if (d <= 32) { constexpr int DP = 32; CALL; }      \
        else if (d <= 64) { constexpr int DP = 64; CALL; } \
        else if (d <= 128) { constexpr int DP = 128; CALL; } \
        else { constexpr int DP = 256; CALL; }             \
    } while (0)
