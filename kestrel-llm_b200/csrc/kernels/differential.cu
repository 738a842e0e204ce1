// Differential attention: a head has two softmax maps over the same values, a1 and a2, and its output is
//
//   o = a1 - lambda a2,   o <- o / sqrt(mean(o^2) + eps) * (1 - diff)
//   lambda = exp(sum(lq1 * lk1)) - exp(sum(lq2 * lk2)) + diff,   one number a layer
//
// The maps' outputs arrive in float32, [T, heads, 2, vd], as the attention kernels write them for 2 * heads query heads whose
// rows are zero outside their own map's part of a cache row (attention_prepare_ex.cu, `maps`).
#include "common.cuh"
#include <math.h>

#define DC_WARPS 4

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

template <typename T>
__global__ void __launch_bounds__(DC_WARPS * 32)
differential_combine_kernel(const float *__restrict__ a, const float *__restrict__ lq1, const float *__restrict__ lk1,
                            const float *__restrict__ lq2, const float *__restrict__ lk2, int dim, float diff, float eps, T *__restrict__ out,
                            int n_heads, int vd) {
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float lam = differential_lambda(lq1, lk1, lq2, lk2, dim, diff, lane);       // weights: not the predecessor's output
    pdl_wait();
    const long long h = (long long)blockIdx.x * DC_WARPS + warp;                      // (token, head)
    if (h >= n_heads) return;
    const float *a1 = a + (size_t)h * 2 * vd, *a2 = a1 + vd;
    float o[8], ss = 0.f;                             // vd <= 256
#pragma unroll
    for (int c = 0; c < 8; ++c) {
        const int i = lane + 32 * c;
        o[c] = i < vd ? a1[i] - lam * a2[i] : 0.f;
        ss = fmaf(o[c], o[c], ss);
    }
    ss = warp_sum(ss);
    const float mul = 1.0f / sqrtf(ss / (float)vd + eps) * (1.0f - diff);
#pragma unroll
    for (int c = 0; c < 8; ++c) {
        const int i = lane + 32 * c;
        if (i < vd) out[(size_t)h * vd + i] = from_f32<T>(o[c] * mul);
    }
}

KESTREL_API int kestrel_differential_combine(const float *a, const float *lq1, const float *lk1, const float *lq2, const float *lk2, int dim,
                                             float diff, float eps, void *out, int dtype, int T, int H, int vd, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && H > 0 && dim > 0 && vd > 0 && vd <= 256 && (long long)T * H < (1ll << 31), "differential_combine: bad sizes");
    const int n = T * H;
    const dim3 grid((n + DC_WARPS - 1) / DC_WARPS);
    if (dtype == KESTREL_F32)
        kestrel_launch(differential_combine_kernel<float>, grid, dim3(DC_WARPS * 32), 0, stream, a, lq1, lk1, lq2, lk2, dim, diff, eps, (float *)out, n, vd);
    else if (dtype == KESTREL_BF16)
        kestrel_launch(differential_combine_kernel<__nv_bfloat16>, grid, dim3(DC_WARPS * 32), 0, stream, a, lq1, lk1, lq2, lk2, dim, diff, eps, (__nv_bfloat16 *)out, n, vd);
    else
        return kestrel_fail(-2, "differential_combine: unknown dtype %d", dtype);
    return kestrel_check_launch("differential_combine");
}
