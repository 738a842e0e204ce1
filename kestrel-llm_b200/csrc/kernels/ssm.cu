// A state-space mixer with a scalar decay per head (Mamba-2).  Per head n, with B and C of its group and a step size dt:
//
//     S_t = exp(-exp(A_log) dt_t) S_{t-1} + dt_t B_t x_t^T,    y_t = S_t^T C_t + D x_t
//
// x | B | C come out of a short convolution (short_conv.cu) as columns of `act`; dt = softplus(logit + dt_bias), float32.  y is
// multiplied by silu(z) and normed in equal parts of the concatenated heads, after the gate.
//
//   expand        what the sequential scan of linear_recurrence.cu takes, head by head: r = C, k = B, v = dt x, w = the decay
//   out           + D x, gate, norm per part, weight, to the storage type
#include "common.cuh"
#include <math.h>

__device__ __forceinline__ float ssm_softplus(float a) { return a > 20.f ? a : log1pf(expf(a)); }

__global__ void __launch_bounds__(256)
ssm_expand_kernel(const float *__restrict__ act, int C, const float *__restrict__ p, int S, size_t slice_stride, int ld, int col_dt,
                  const float *__restrict__ dt_bias, const float *__restrict__ A_log, float *__restrict__ r_out, float *__restrict__ w_out,
                  float *__restrict__ k_out, float *__restrict__ v_out, int H, int G, int N, int P) {
    extern __shared__ float ssm_dt[];                         // [H] step sizes, [H] decays
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, inner = H * P;
    for (int h = threadIdx.x; h < H; h += 256) {
        const float dt = ssm_softplus(sum_slices(p, S, slice_stride, (size_t)t * ld + col_dt + h) + dt_bias[h]);
        ssm_dt[h] = dt;
        ssm_dt[H + h] = expf(-expf(A_log[h]) * dt);
    }
    __syncthreads();
    const float *a = act + (size_t)t * C;
    for (int i = threadIdx.x; i < H * N; i += 256) {
        const int h = i / N, g = h / (H / G), c = g * N + i % N;
        const size_t o = (size_t)t * H * N + i;
        k_out[o] = a[inner + c];
        r_out[o] = a[inner + G * N + c];
        w_out[o] = ssm_dt[H + h];
    }
    for (int i = threadIdx.x; i < inner; i += 256) v_out[(size_t)t * inner + i] = ssm_dt[i / P] * a[i];
}

KESTREL_API int kestrel_ssm_expand(const float *act, const float *partial, int S, long long slice_stride, int ld, int col_dt, const float *dt_bias,
                                   const float *A_log, float *r_out, float *w_out, float *k_out, float *v_out, int T, int H, int G, int N, int P,
                                   cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && S > 0 && H > 0 && G > 0 && H % G == 0 && N > 0 && P > 0 && H <= 4096 && col_dt >= 0 && col_dt + H <= ld, "ssm_expand: bad sizes");
    kestrel_launch(ssm_expand_kernel, dim3(T), dim3(256), 2 * (size_t)H * sizeof(float), stream, act, H * P + 2 * G * N, partial, S, (size_t)slice_stride, ld,
                   col_dt, dt_bias, A_log, r_out, w_out, k_out, v_out, H, G, N, P);
    return kestrel_check_launch("ssm_expand");
}

// o [T, H P] = S^T C; y = (o + D x) silu(z), normed in `parts` equal parts.  A block a (token, part).
template <typename T>
__global__ void __launch_bounds__(256)
ssm_out_kernel(const float *__restrict__ o, const float *__restrict__ act, int C, const float *__restrict__ D, const float *__restrict__ p, int S,
               size_t slice_stride, int ld, int col_z, const float *__restrict__ w, float eps, T *__restrict__ out, int inner, int parts, int P) {
    extern __shared__ float ssm_y[];
    __shared__ float red[8];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, n = inner / parts, c0 = blockIdx.y * n, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += 256) {
        const int c = c0 + i;
        const float z = sum_slices(p, S, slice_stride, (size_t)t * ld + col_z + c);
        const float y = fmaf(D[c / P], act[(size_t)t * C + c], o[(size_t)t * inner + c]) * (z / (1.0f + expf(-z)));
        ssm_y[i] = y;
        ss = fmaf(y, y, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) tot += red[k];
    const float mul = 1.0f / sqrtf(tot / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += 256) out[(size_t)t * inner + c0 + i] = from_f32<T>(ssm_y[i] * mul * w[c0 + i]);
}

KESTREL_API int kestrel_ssm_out(const float *o, const float *act, const float *D, const float *partial, int S, long long slice_stride, int ld, int col_z,
                                const float *w, float eps, void *out, int dtype, int T, int H, int G, int N, int P, int parts, cudaStream_t stream) {
    if (T == 0) return 0;
    const int inner = H * P, C = inner + 2 * G * N;
    KESTREL_REQUIRE(T > 0 && S > 0 && H > 0 && P > 0 && parts > 0 && inner % parts == 0 && col_z >= 0 && col_z + inner <= ld, "ssm_out: bad sizes");
    const size_t smem = (size_t)(inner / parts) * sizeof(float);
    KESTREL_REQUIRE(smem <= KESTREL_SMEM_MAX_DYNAMIC - 1024, "ssm_out: %d channels a norm part", inner / parts);
#define SO_GO(TT)                                                                                                                     \
    {                                                                                                                                 \
        static bool attr_set = false;                                                                                                 \
        if (!attr_set && cudaFuncSetAttribute(ssm_out_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, KESTREL_SMEM_MAX_DYNAMIC - 1024) != cudaSuccess) \
            return kestrel_fail(-3, "ssm_out: cannot set the shared memory size");                                                    \
        attr_set = true;                                                                                                              \
        kestrel_launch(ssm_out_kernel<TT>, dim3(T, parts), dim3(256), smem, stream, o, act, C, D, partial, S, (size_t)slice_stride, ld, col_z, w, eps, \
                       (TT *)out, inner, parts, P);                                                                                   \
    }
    if (dtype == KESTREL_F32) SO_GO(float)
    else if (dtype == KESTREL_BF16) SO_GO(__nv_bfloat16)
    else return kestrel_fail(-2, "ssm_out: unknown dtype %d", dtype);
#undef SO_GO
    return kestrel_check_launch("ssm_out");
}
