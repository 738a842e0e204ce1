// Pieces of the kernels that do everything between two products for a step of few tokens: a CTA takes a (request, head), its threads the
// head's state - VEC neighbouring value columns and every groups-th key channel each.
#pragma once
#include "common.cuh"

#define RST_THREADS 256

struct RstLayout {
    int cols, groups, rg, c0;
};
template <int VEC> __device__ __forceinline__ RstLayout rst_layout(int dv) {
    RstLayout l;
    l.cols = dv / VEC;
    l.groups = RST_THREADS / l.cols;
    l.rg = threadIdx.x / l.cols;
    l.c0 = threadIdx.x % l.cols * VEC;
    return l;
}
template <int VEC> __device__ __forceinline__ void rst_load(float (&s)[VEC], const float *p) {
    if constexpr (VEC == 4) {
        const float4 v = *reinterpret_cast<const float4 *>(p);
        s[0] = v.x; s[1] = v.y; s[2] = v.z; s[3] = v.w;
    } else {
        s[0] = p[0];
    }
}
template <int VEC> __device__ __forceinline__ void rst_store(float *p, const float (&s)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4 *>(p) = make_float4(s[0], s[1], s[2], s[3]);
    else p[0] = s[0];
}
// the sum of x over the block, to every thread; red: one float a warp, free to be rewritten after the next barrier
__device__ __forceinline__ float rst_block_sum(float x, float *red) {
    x = warp_sum(x);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = x;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < RST_THREADS / 32; ++w) tot += red[w];
    return tot;
}
// A column's causal convolution at token t of a step (first: the request's first token of it): inputs before that from the request's
// tail [taps - 1][C] at channel c of the filter w [taps][C], which is the product's column col.
__device__ __forceinline__ float rst_conv(const float *__restrict__ p, int S, size_t slice_stride, int ld, int col, const float *__restrict__ w, int taps,
                                          const float *__restrict__ tail, int C, int c, int first, int t) {
    float y = 0.f;
    for (int j = 0; j < taps; ++j) {
        const int n = t - first - (taps - 1) + j;
        const float x = n >= 0 ? sum_slices(p, S, slice_stride, (size_t)(first + n) * ld + col) : tail[(size_t)(taps - 1 + n) * C + c];
        y = fmaf(w[(size_t)j * C + c], x, y);
    }
    return y;
}
