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
// in base-2 units, sum); a slice without visible keys holds zeros, minus infinity and a sum of zero.  Slices in ascending order,
// then the head as above.  A block of 256 threads a (token, head), 128 a map; a column's slices are fetched before their factors
// are known, so that the two round trips overlap.
#define DM_SLICES 64
#define DM_AHEAD 16
__global__ void __launch_bounds__(256)
differential_merge_kernel(const float *__restrict__ part_o, const float *__restrict__ part_ml, int slices, int ld, const DifferentialOpts opts,
                          __nv_bfloat16 *__restrict__ out, int vd) {
    pdl_launch_dependents();
    __shared__ float a_s[2][256], f_s[2][DM_SLICES + 1];
    __shared__ float red[8];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const float lam = differential_lambda(opts, lane);
    pdl_wait();
    const size_t h = blockIdx.x;                      // (token, head)
    const int map = tid >> 7, c0 = tid & 127;
    const size_t row = (h * 2 + map) * slices;
    float x[DM_AHEAD];
#pragma unroll
    for (int s = 0; s < DM_AHEAD; ++s) x[s] = s < slices && c0 < vd ? part_o[(row + s) * ld + c0] : 0.f;
    if ((warp & 3) == 0) {
        // the slices' factors 2^(m_s - M), a lane a slice and another 32 further on, and the row's sum
        float m[2], l[2];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int s = lane + 32 * k;
            const float2 ml = s < slices ? *reinterpret_cast<const float2 *>(part_ml + (row + s) * 2) : make_float2(-INFINITY, 0.f);
            m[k] = ml.x;
            l[k] = ml.y;
        }
        const float M = warp_max(fmaxf(m[0], m[1]));
        float L = 0.f;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float f = m[k] == -INFINITY ? 0.f : exp2f(m[k] - M);
            f_s[map][lane + 32 * k] = f;
            L = fmaf(l[k], f, L);
        }
        L = warp_sum(L);
        if (lane == 0) f_s[map][DM_SLICES] = 1.0f / L;
    }
    __syncthreads();
    for (int c = c0; c < vd; c += 128) {
        float acc = 0.f;
        if (c == c0) {
#pragma unroll
            for (int s = 0; s < DM_AHEAD; ++s) acc = fmaf(x[s], s < slices ? f_s[map][s] : 0.f, acc);
#pragma unroll 4
            for (int s = DM_AHEAD; s < slices; ++s) acc = fmaf(part_o[(row + s) * ld + c], f_s[map][s], acc);
        } else {
#pragma unroll 8
            for (int s = 0; s < slices; ++s) acc = fmaf(part_o[(row + s) * ld + c], f_s[map][s], acc);
        }
        a_s[map][c] = acc * f_s[map][DM_SLICES];
    }
    __syncthreads();
    const float o = tid < vd ? a_s[0][tid] - lam * a_s[1][tid] : 0.f;      // vd <= 256
    const float ss = warp_sum(o * o);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) tot += red[k];
    if (tid < vd) out[h * vd + tid] = __float2bfloat16_rn(o * (1.0f / sqrtf(tot / (float)vd + opts.eps) * (1.0f - opts.diff)));
}

KESTREL_API int kestrel_differential_merge(const float *part_o, const float *part_ml, int slices, int ld, const float *lq1, const float *lk1,
                                           const float *lq2, const float *lk2, int dim, float diff, float eps, void *out, int T, int H, int vd,
                                           cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && H > 0 && slices > 0 && slices <= DM_SLICES && dim > 0 && vd > 0 && vd <= 256 && ld >= vd && (long long)T * H < (1ll << 31), "differential_merge: bad sizes");
    const DifferentialOpts opts = {lq1, lk1, lq2, lk2, dim, diff, eps};
    kestrel_launch(differential_merge_kernel, dim3(T * H), dim3(256), 0, stream, part_o, part_ml, slices, ld, opts, (__nv_bfloat16 *)out, vd);
    return kestrel_check_launch("differential_merge");
}
