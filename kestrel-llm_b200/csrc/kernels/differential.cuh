// What the kernels of differential attention share: a layer's constants and its weight of the second map.
#pragma once
#include "common.cuh"
#include <math.h>

struct DifferentialOpts {
    const float *lq1, *lk1, *lq2, *lk2;      // [dim]
    int dim;
    float diff, eps;
};

// lambda, the same bits in every warp: the sums run over the lanes' elements in ascending order, then a shuffle tree
__device__ __forceinline__ float differential_lambda(const float *lq1, const float *lk1, const float *lq2, const float *lk2, int dim, float diff,
                                                     int lane) {
    float a = 0.f, b = 0.f;
    for (int i = lane; i < dim; i += 32) {
        a = fmaf(lq1[i], lk1[i], a);
        b = fmaf(lq2[i], lk2[i], b);
    }
    return expf(warp_sum(a)) - expf(warp_sum(b)) + diff;
}
__device__ __forceinline__ float differential_lambda(const DifferentialOpts &o, int lane) {
    return differential_lambda(o.lq1, o.lk1, o.lq2, o.lk2, o.dim, o.diff, lane);
}
