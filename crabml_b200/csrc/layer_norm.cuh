// layer_norm.cuh -- the layer norm of one row by one CTA, shared by the plain op (seqops.cu) and by the products that norm their own input
// (parallel_block.cu).
#pragma once
#include "common.cuh"

#define LN_KEEP 8
template <int THREADS>
__device__ __forceinline__ float ln_block_sum(float v, float* red) {
    v = warp_sum(v);
    __syncthreads();                                         // red may still be read from the sum before
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; w++) t += red[w];
    return t;
}
// A thread keeps its (up to LN_KEEP) elements of the row in registers, so the row is read once; the mean first (thread-strided partial sums,
// the butterfly, then the warps' sums in warp order), then the mean of the squared deviations from it in the same order, then
// store(column, (x - mean) / sqrt(var + eps) * w + b) for every column.  The order depends on the row's length and THREADS alone.
// red: THREADS / 32 floats of shared memory.  store may overwrite the row: thread t only ever touches columns t, t + THREADS, ...
template <int THREADS, class Store>
__device__ __forceinline__ void layer_norm_row(const float* xr, const float* __restrict__ w, const float* __restrict__ b, int cols, float eps, float* red, Store store) {
    float keep[LN_KEEP];
    float s = 0.0f;
#pragma unroll
    for (int e = 0; e < LN_KEEP; e++) {
        const int c = threadIdx.x + e * THREADS;
        keep[e] = c < cols ? xr[c] : 0.0f;
        s += keep[e];
    }
    for (int c = threadIdx.x + LN_KEEP * THREADS; c < cols; c += THREADS) s += xr[c];
    const float mean = ln_block_sum<THREADS>(s, red) / (float)cols;
    float ss = 0.0f;
#pragma unroll
    for (int e = 0; e < LN_KEEP; e++) {
        const int c = threadIdx.x + e * THREADS;
        const float d = keep[e] - mean;
        if (c < cols) ss = fmaf(d, d, ss);
    }
    for (int c = threadIdx.x + LN_KEEP * THREADS; c < cols; c += THREADS) { const float d = xr[c] - mean; ss = fmaf(d, d, ss); }
    const float inv = 1.0f / sqrtf(ln_block_sum<THREADS>(ss, red) / (float)cols + eps);
#pragma unroll
    for (int e = 0; e < LN_KEEP; e++) {
        const int c = threadIdx.x + e * THREADS;
        if (c < cols) { const float v = (keep[e] - mean) * inv * w[c]; store(c, b ? v + b[c] : v); }
    }
    for (int c = threadIdx.x + LN_KEEP * THREADS; c < cols; c += THREADS) { const float v = (xr[c] - mean) * inv * w[c]; store(c, b ? v + b[c] : v); }
}
