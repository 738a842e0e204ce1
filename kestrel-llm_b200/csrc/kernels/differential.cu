// Differential attention: a head has two softmax maps over the same values, a1 and a2, and its output is
//
//   o = a1 - lambda a2,   o <- o / sqrt(mean(o^2) + eps) * (1 - diff)
//   lambda = exp(sum(lq1 * lk1)) - exp(sum(lq2 * lk2)) + diff,   one number a layer
//
// The maps' outputs arrive in float32, [T, heads, 2, vd], as the attention kernels write them for 2 * heads query heads whose
// rows are zero outside their own map's part of a cache row (attention_prepare_ex.cu, `maps`).
#include "common.cuh"
#include "differential.cuh"
#include <math.h>

#define DC_WARPS 4

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

// The maps' outputs as key-range slices: part_o [T * H * 2, slices, ld] unnormalised, part_ml [T * H * 2, slices, 2] the slices' (maximum
// in base-2 units, sum).  Slices in ascending order, then the head as above.  A block of four warps a (token, head): warps 0, 1
// first merge map 1, warps 2, 3 map 2, each its half of the columns.
#define DM_SLICES 64
__global__ void __launch_bounds__(128)
differential_merge_kernel(const float *__restrict__ part_o, const float *__restrict__ part_ml, int slices, int ld, const DifferentialOpts opts,
                          __nv_bfloat16 *__restrict__ out, int vd) {
    pdl_launch_dependents();
    __shared__ float a_s[2][256], f_s[2][DM_SLICES + 1];
    __shared__ float red[4];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const float lam = differential_lambda(opts, lane);
    pdl_wait();
    const size_t h = blockIdx.x;                      // (token, head)
    const int map = tid >> 6;
    const size_t row = (h * 2 + map) * slices;
    if ((warp & 1) == 0) {
        // the slices' factors 2^(m_s - M), a lane a slice (further ones in rounds), and the row's sum in ascending order
        float M = -INFINITY, L = 0.f;
        for (int s = lane; s < slices; s += 32) M = fmaxf(M, part_ml[(row + s) * 2]);
        M = warp_max(M);
        for (int s0 = 0; s0 < slices; s0 += 32) {
            const int s = s0 + lane;
            const float m = s < slices ? part_ml[(row + s) * 2] : -INFINITY, f = m == -INFINITY ? 0.f : exp2f(m - M);
            const float l = s < slices && f > 0.f ? part_ml[(row + s) * 2 + 1] * f : 0.f;
            if (s < slices && s < DM_SLICES) f_s[map][s] = f;
            for (int k = 0; k < min(32, slices - s0); ++k) L += __shfl_sync(0xffffffffu, l, k);
        }
        if (lane == 0) f_s[map][DM_SLICES] = 1.0f / L;
    }
    __syncthreads();
    for (int c = tid & 63; c < vd; c += 64) {
        float acc = 0.f;
#pragma unroll 8
        for (int s = 0; s < slices; ++s)
            if (f_s[map][s] > 0.f) acc = fmaf(part_o[(row + s) * ld + c], f_s[map][s], acc);
        a_s[map][c] = acc * f_s[map][DM_SLICES];
    }
    __syncthreads();
    float o[2], ss = 0.f;                             // vd <= 256
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const int c = tid + 128 * k;
        o[k] = c < vd ? a_s[0][c] - lam * a_s[1][c] : 0.f;
        ss = fmaf(o[k], o[k], ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    const float mul = 1.0f / sqrtf(((red[0] + red[1]) + (red[2] + red[3])) / (float)vd + opts.eps) * (1.0f - opts.diff);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const int c = tid + 128 * k;
        if (c < vd) out[h * vd + c] = __float2bfloat16_rn(o[k] * mul);
    }
}

KESTREL_API int kestrel_differential_merge(const float *part_o, const float *part_ml, int slices, int ld, const float *lq1, const float *lk1,
                                           const float *lq2, const float *lk2, int dim, float diff, float eps, void *out, int T, int H, int vd,
                                           cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && H > 0 && slices > 0 && slices <= DM_SLICES && dim > 0 && vd > 0 && vd <= 256 && ld >= vd && (long long)T * H < (1ll << 31), "differential_merge: bad sizes");
    const DifferentialOpts opts = {lq1, lk1, lq2, lk2, dim, diff, eps};
    kestrel_launch(differential_merge_kernel, dim3(T * H), dim3(128), 0, stream, part_o, part_ml, slices, ld, opts, (__nv_bfloat16 *)out, vd);
    return kestrel_check_launch("differential_merge");
}
