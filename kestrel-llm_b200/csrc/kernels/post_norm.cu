// A norm on a sublayer's result and the add to the stream, vectorised, for rows whose length is a multiple of 4:
//
//   residual[t] += y / sqrt(mean(y^2) + eps) * w,     copy[t] = residual[t] in the storage type (where a copy is given)
//
// or, with a second weight, copy[t] = the norm of the new residual[t]: the input of the sublayer that follows.
//
// with y either a product (float32 slices in ascending order, plus a bias) or the sum of a routed feed-forward that was never
// written out (`MoeSource`): the chosen experts' weighted rows in the order of choice, the identity experts' weights times
// the input row, and an expert that every token takes times its gate.  A block takes a row, its threads the row's float4s; the
// sum of squares is a fixed tree over the row's length alone, so a row's bits do not depend on the step.
#include "common.cuh"
#include <math.h>

struct ProductSource {
    const float *y;
    int S;
    size_t stride;
    const float *bias;
};

struct MoeSource {
    const float *y;                      // [rows sorted by expert, d], weighted
    const int *pair_row, *ids;           // [T, top]
    const float *weights;                // [T, top]
    int top, experts;
    const void *x;                       // the input rows, in the copy's type
    long long ldx;
    const float *shared;                 // slices, or null
    int Ss;
    size_t shared_stride;
    const float *z;                      // the product whose column sg_col is the shared expert's gate, or null
    int Sz;
    size_t z_stride;
    int z_ld, sg_col;
};

__device__ __forceinline__ void pn_add(float4 &v, const float4 x) { v.x += x.x; v.y += x.y; v.z += x.z; v.w += x.w; }
__device__ __forceinline__ void pn_fma(float4 &v, float a, const float4 x) {
    v.x = fmaf(a, x.x, v.x); v.y = fmaf(a, x.y, v.y); v.z = fmaf(a, x.z, v.z); v.w = fmaf(a, x.w, v.w);
}
__device__ __forceinline__ float4 pn_load(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 pn_load(const __nv_bfloat16 *p) {
    const uint2 u = *reinterpret_cast<const uint2 *>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162 *>(&u.x), b = *reinterpret_cast<const __nv_bfloat162 *>(&u.y);
    return make_float4(__bfloat162float(a.x), __bfloat162float(a.y), __bfloat162float(b.x), __bfloat162float(b.y));
}
__device__ __forceinline__ void pn_store(float *p, const float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void pn_store(__nv_bfloat16 *p, const float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<uint32_t *>(&a), *reinterpret_cast<uint32_t *>(&b));
}

#define PN_MAX_THREADS 512
#define PN_MAX_TOP 32

template <typename T, int NV, typename Source>
__global__ void __launch_bounds__(PN_MAX_THREADS)
post_norm_kernel(float *__restrict__ residual, const Source src, const float *__restrict__ w, float eps, T *__restrict__ copy,
                 const float *__restrict__ next_w, float next_eps, int d) {
    constexpr bool MOE = sizeof(Source) == sizeof(MoeSource);
    pdl_launch_dependents();
    __shared__ float red[PN_MAX_THREADS / 32];
    __shared__ int row_s[PN_MAX_TOP];                 // MOE: the rows of the token's experts, -1 for an identity expert
    __shared__ float direct_s, gate_s;
    const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31;
    float4 v[NV], g[NV], gn[NV];
#pragma unroll
    for (int c = 0; c < NV; ++c) {                    // weights: before the wait
        const int i = 4 * (tid + c * nt);
        g[c] = i < d ? pn_load(w + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        gn[c] = next_w && i < d ? pn_load(next_w + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if constexpr (MOE) {
        pdl_wait();
        if (tid < 32) {
            const bool in = tid < src.top;
            const int id = in ? src.ids[(size_t)t * src.top + tid] : 0;
            row_s[tid] = in && id < src.experts ? src.pair_row[(size_t)t * src.top + tid] : -1;
            const float sum = warp_sum(in && id >= src.experts ? src.weights[(size_t)t * src.top + tid] : 0.f);
            if (tid == 0) {
                direct_s = sum;
                gate_s = src.z ? 1.0f / (1.0f + expf(-sum_slices(src.z, src.Sz, src.z_stride, (size_t)t * src.z_ld + src.sg_col))) : 1.0f;
            }
        }
        __syncthreads();
        const float direct = direct_s, gate = gate_s;
        float4 e[NV], sh[NV];
#pragma unroll
        for (int c = 0; c < NV; ++c) v[c] = e[c] = sh[c] = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int k = 0; k < src.top; ++k) {
            const int row = row_s[k];
            if (row < 0) continue;
#pragma unroll
            for (int c = 0; c < NV; ++c) {
                const int i = 4 * (tid + c * nt);
                if (i < d) pn_add(v[c], pn_load(src.y + (size_t)row * d + i));
            }
        }
        if (src.shared) {
            for (int s = 0; s < src.Ss; ++s)
#pragma unroll
                for (int c = 0; c < NV; ++c) {
                    const int i = 4 * (tid + c * nt);
                    if (i < d) pn_add(sh[c], pn_load(src.shared + (size_t)s * src.shared_stride + (size_t)t * d + i));
                }
        }
#pragma unroll
        for (int c = 0; c < NV; ++c) {
            const int i = 4 * (tid + c * nt);
            if (i >= d) continue;
            if (direct != 0.f) pn_fma(v[c], direct, pn_load((const T *)src.x + (size_t)t * src.ldx + i));
            if (src.shared) pn_fma(v[c], gate, sh[c]);
        }
    } else {
        float4 b[NV];
#pragma unroll
        for (int c = 0; c < NV; ++c) {                // the bias is a weight: before the wait
            const int i = 4 * (tid + c * nt);
            b[c] = src.bias && i < d ? pn_load(src.bias + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            v[c] = make_float4(0.f, 0.f, 0.f, 0.f);
        }
        pdl_wait();
#pragma unroll 8
        for (int s = 0; s < src.S; ++s)
#pragma unroll
            for (int c = 0; c < NV; ++c) {
                const int i = 4 * (tid + c * nt);
                if (i < d) pn_add(v[c], pn_load(src.y + (size_t)s * src.stride + (size_t)t * d + i));
            }
#pragma unroll
        for (int c = 0; c < NV; ++c) pn_add(v[c], b[c]);
    }
    float4 x[NV];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < NV; ++c) {
        const int i = 4 * (tid + c * nt);
        x[c] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i >= d) continue;
        x[c] = pn_load(residual + (size_t)t * d + i);
        ss = fmaf(v[c].x, v[c].x, fmaf(v[c].y, v[c].y, fmaf(v[c].z, v[c].z, fmaf(v[c].w, v[c].w, ss))));
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int k = 0; k < nt / 32; ++k) tot += red[k];
    const float mul = 1.0f / sqrtf(tot / (float)d + eps);
#pragma unroll
    for (int c = 0; c < NV; ++c) {
        const int i = 4 * (tid + c * nt);
        if (i >= d) continue;
        x[c].x += v[c].x * mul * g[c].x;
        x[c].y += v[c].y * mul * g[c].y;
        x[c].z += v[c].z * mul * g[c].z;
        x[c].w += v[c].w * mul * g[c].w;
        pn_store(residual + (size_t)t * d + i, x[c]);
        if (copy && !next_w) pn_store(copy + (size_t)t * d + i, x[c]);
    }
    if (!next_w) return;
    ss = 0.f;
#pragma unroll
    for (int c = 0; c < NV; ++c) {
        const int i = 4 * (tid + c * nt);
        if (i >= d) continue;
        ss = fmaf(x[c].x, x[c].x, fmaf(x[c].y, x[c].y, fmaf(x[c].z, x[c].z, fmaf(x[c].w, x[c].w, ss))));
    }
    ss = warp_sum(ss);
    __syncthreads();                                  // everyone has read the first sums
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    tot = 0.f;
    for (int k = 0; k < nt / 32; ++k) tot += red[k];
    const float mul2 = 1.0f / sqrtf(tot / (float)d + next_eps);
#pragma unroll
    for (int c = 0; c < NV; ++c) {
        const int i = 4 * (tid + c * nt);
        if (i >= d) continue;
        pn_store(copy + (size_t)t * d + i, make_float4(x[c].x * mul2 * gn[c].x, x[c].y * mul2 * gn[c].y, x[c].z * mul2 * gn[c].z, x[c].w * mul2 * gn[c].w));
    }
}

template <typename T, typename Source>
static int pn_launch(float *residual, const Source &src, const float *w, float eps, T *copy, int n_tokens, int d, cudaStream_t stream,
                     const float *next_w = nullptr, float next_eps = 0.f) {
    int nt = (d / 4 + 31) / 32 * 32;
    if (nt > PN_MAX_THREADS) nt = PN_MAX_THREADS;
    const int nv = (d / 4 + nt - 1) / nt;
#define PN_CASE(N) kestrel_launch(post_norm_kernel<T, N, Source>, dim3(n_tokens), dim3(nt), 0, stream, residual, src, w, eps, copy, next_w, next_eps, d)
    if (nv <= 1) PN_CASE(1);
    else if (nv <= 2) PN_CASE(2);
    else if (nv <= 4) PN_CASE(4);
    else PN_CASE(8);
#undef PN_CASE
    return kestrel_check_launch("post_norm");
}

// whether the kernels take rows of d numbers
KESTREL_API int kestrel_post_norm_takes(int d) { return d > 0 && d % 4 == 0 && d <= 4 * PN_MAX_THREADS * 8; }

KESTREL_API int kestrel_post_norm_add(float *residual, const float *y, int S, long long stride, const float *bias, const float *w, float eps, void *copy,
                                      int dtype, int T, int d, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && S > 0 && kestrel_post_norm_takes(d) && stride % 4 == 0, "post_norm_add: bad sizes T=%d d=%d", T, d);
    const ProductSource src = {y, S, (size_t)stride, bias};
    if (dtype == KESTREL_F32) return pn_launch<float>(residual, src, w, eps, (float *)copy, T, d, stream);
    if (dtype == KESTREL_BF16) return pn_launch<__nv_bfloat16>(residual, src, w, eps, (__nv_bfloat16 *)copy, T, d, stream);
    return kestrel_fail(-2, "post_norm_add: unknown dtype %d", dtype);
}

// copy[t] = the norm of the new residual[t] with the weight next_w
KESTREL_API int kestrel_post_norm_add_norm(float *residual, const float *y, int S, long long stride, const float *bias, const float *w, float eps,
                                           const float *next_w, float next_eps, void *copy, int dtype, int T, int d, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && S > 0 && kestrel_post_norm_takes(d) && stride % 4 == 0 && next_w && copy, "post_norm_add_norm: bad sizes T=%d d=%d", T, d);
    const ProductSource src = {y, S, (size_t)stride, bias};
    if (dtype == KESTREL_F32) return pn_launch<float>(residual, src, w, eps, (float *)copy, T, d, stream, next_w, next_eps);
    if (dtype == KESTREL_BF16) return pn_launch<__nv_bfloat16>(residual, src, w, eps, (__nv_bfloat16 *)copy, T, d, stream, next_w, next_eps);
    return kestrel_fail(-2, "post_norm_add_norm: unknown dtype %d", dtype);
}

KESTREL_API int kestrel_post_norm_add_moe(float *residual, const float *y, const int *pair_row, const int *ids, const float *weights, int top, int experts,
                                          const void *x, long long ldx, const float *shared, int Ss, long long shared_stride, const float *z, int Sz,
                                          long long z_stride, int z_ld, int sg_col, const float *w, float eps, void *copy, int dtype, int T, int d,
                                          cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && top > 0 && top <= PN_MAX_TOP && experts >= 0 && kestrel_post_norm_takes(d) && shared_stride % 4 == 0 && ldx % 4 == 0 &&
                    (!shared || Ss > 0) && (!z || (Sz > 0 && sg_col >= 0 && sg_col < z_ld)), "post_norm_add_moe: bad sizes T=%d d=%d", T, d);
    const MoeSource src = {y, pair_row, ids, weights, top, experts, x, ldx, shared, Ss, (size_t)shared_stride, z, Sz, (size_t)z_stride, z_ld, sg_col};
    if (dtype == KESTREL_F32) return pn_launch<float>(residual, src, w, eps, (float *)copy, T, d, stream);
    if (dtype == KESTREL_BF16) return pn_launch<__nv_bfloat16>(residual, src, w, eps, (__nv_bfloat16 *)copy, T, d, stream);
    return kestrel_fail(-2, "post_norm_add_moe: unknown dtype %d", dtype);
}

// x[t] = table[ids[t]] in float32 and copy[t] = the same row as the table holds it: the start of a stream whose first sublayer reads
// it unnormed
__global__ void __launch_bounds__(256)
embed_copy_kernel(const __nv_bfloat16 *__restrict__ table, const int *__restrict__ ids, float *__restrict__ x, __nv_bfloat16 *__restrict__ copy, int d) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const uint2 *row = reinterpret_cast<const uint2 *>(table + (size_t)ids[t] * d);
    for (int i = threadIdx.x; i < d / 4; i += blockDim.x) {
        const uint2 u = row[i];
        *reinterpret_cast<uint2 *>(copy + (size_t)t * d + 4 * i) = u;
        pn_store(x + (size_t)t * d + 4 * i, pn_load(reinterpret_cast<const __nv_bfloat16 *>(row + i)));
    }
}

KESTREL_API int kestrel_embed_copy(const void *table, const int *ids, float *x, void *copy, int T, int d, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && d > 0 && d % 4 == 0, "embed_copy: bad sizes T=%d d=%d", T, d);
    kestrel_launch(embed_copy_kernel, dim3(T), dim3(256), 0, stream, (const __nv_bfloat16 *)table, ids, x, (__nv_bfloat16 *)copy, d);
    return kestrel_check_launch("embed_copy");
}
