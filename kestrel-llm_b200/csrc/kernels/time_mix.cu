// A recurrence whose projections read each token blended with the one before it (the RWKV form of linear attention).
//
//   token_shift   mixes[s][t] = h[t] + (h[t - 1] - h[t]) * mu[s], s = 0 .. n - 1: the inputs of n projections.  The token before a
//                 request's first one of this step comes from its state slot (zeros for a new request)
//   gates         r, k, v out of their products' slices; w = exp(-exp(z + w0)), the decay per head and key channel, float32; and
//                 the request's last h of this step into its state slot (every reader of the old one is done by then)
//   scan          linear_recurrence.cu, the form that reads the old state with a bonus for the token's own write
//   (output)      head_norm_act: per-head norm, weight, silu of the gate's product
#include "common.cuh"
#include "recurrence_step.cuh"
#include <math.h>

template <typename T> struct TmVec;
template <> struct TmVec<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(float (&x)[4], const float *p) { const float4 v = *reinterpret_cast<const float4 *>(p); x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w; }
    static __device__ __forceinline__ void store(float *p, const float (&x)[4]) { *reinterpret_cast<float4 *>(p) = make_float4(x[0], x[1], x[2], x[3]); }
};
template <> struct TmVec<__nv_bfloat16> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(float (&x)[4], const __nv_bfloat16 *p) {
        const uint2 u = *reinterpret_cast<const uint2 *>(p);
        const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162 *>(&u.x), b = *reinterpret_cast<const __nv_bfloat162 *>(&u.y);
        x[0] = __bfloat162float(a.x); x[1] = __bfloat162float(a.y); x[2] = __bfloat162float(b.x); x[3] = __bfloat162float(b.y);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16 *p, const float (&x)[4]) {
        __nv_bfloat162 a = __floats2bfloat162_rn(x[0], x[1]), b = __floats2bfloat162_rn(x[2], x[3]);
        *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<uint32_t *>(&a), *reinterpret_cast<uint32_t *>(&b));
    }
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
token_shift_kernel(const T *__restrict__ h, const float *__restrict__ mu, int n, const float *__restrict__ state, size_t state_stride, size_t state_off,
                   const int *__restrict__ seq_of_token, const int *__restrict__ cu_seqlens, const int *__restrict__ slots, T *__restrict__ out, int n_tokens,
                   int d) {
    constexpr int V = VEC ? TmVec<T>::N : 1;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, seq = seq_of_token[t];
    const bool in_step = t > cu_seqlens[seq];
    const float *kept = state + (size_t)slots[seq] * state_stride + state_off;
    for (int i = (blockIdx.y * 256 + threadIdx.x) * V; i < d; i += gridDim.y * 256 * V) {
        float x[V], before[V];
        if constexpr (VEC) {
            TmVec<T>::load(x, h + (size_t)t * d + i);
            if (in_step) TmVec<T>::load(before, h + (size_t)(t - 1) * d + i);
            else TmVec<float>::load(before, kept + i);
        } else {
            x[0] = to_f32<T>(h[(size_t)t * d + i]);
            before[0] = in_step ? to_f32<T>(h[(size_t)(t - 1) * d + i]) : kept[i];
        }
        for (int s = 0; s < n; ++s) {
            float y[V];
            if constexpr (VEC) {
                float m[V];
                TmVec<float>::load(m, mu + (size_t)s * d + i);
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] = fmaf(before[e] - x[e], m[e], x[e]);
                TmVec<T>::store(out + ((size_t)s * n_tokens + t) * d + i, y);
            } else {
                y[0] = fmaf(before[0] - x[0], mu[(size_t)s * d + i], x[0]);
                out[((size_t)s * n_tokens + t) * d + i] = from_f32<T>(y[0]);
            }
        }
    }
}

KESTREL_API int kestrel_token_shift(const void *h, const float *mu, int n, const float *state, long long state_stride, long long state_off,
                                    const int *seq_of_token, const int *cu_seqlens, const int *slots, void *out, int dtype, int T, int d,
                                    cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && d > 0 && n > 0 && state_off >= 0, "token_shift: bad sizes");
    const bool vec = d % 4 == 0 && state_stride % 4 == 0 && state_off % 4 == 0 && (((uintptr_t)h | (uintptr_t)out | (uintptr_t)mu | (uintptr_t)state) & 15) == 0;
    const dim3 grid(T, T >= 256 ? 1 : (d + 1023) / 1024);
#define TM_GO(TT, V) kestrel_launch(token_shift_kernel<TT, V>, grid, dim3(256), 0, stream, (const TT *)h, mu, n, state, (size_t)state_stride, (size_t)state_off, \
                                    seq_of_token, cu_seqlens, slots, (TT *)out, T, d)
    if (dtype == KESTREL_F32) { if (vec) TM_GO(float, true); else TM_GO(float, false); }
    else if (dtype == KESTREL_BF16) { if (vec) TM_GO(__nv_bfloat16, true); else TM_GO(__nv_bfloat16, false); }
    else return kestrel_fail(-2, "token_shift: unknown dtype %d", dtype);
#undef TM_GO
    return kestrel_check_launch("token_shift");
}

// r, k, v: columns 0, n, 2 n of the product p; the decay's logits: the product z [T, n]
template <typename T>
__global__ void __launch_bounds__(256)
time_mix_gates_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, const float *__restrict__ z, int Sz, size_t z_stride,
                      const float *__restrict__ w0, float *__restrict__ r_out, float *__restrict__ k_out, float *__restrict__ v_out,
                      float *__restrict__ w_out, int n, const T *__restrict__ h, int d, float *__restrict__ state, size_t state_stride, size_t state_off,
                      const int *__restrict__ seq_of_token, const int *__restrict__ cu_seqlens, const int *__restrict__ slots) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, seq = seq_of_token[t];
    const size_t row = (size_t)t * ld;
    for (int i = blockIdx.y * 256 + threadIdx.x; i < n; i += gridDim.y * 256) {
        const size_t o = (size_t)t * n + i;
        r_out[o] = sum_slices(p, S, slice_stride, row + i);
        k_out[o] = sum_slices(p, S, slice_stride, row + n + i);
        v_out[o] = sum_slices(p, S, slice_stride, row + 2 * (size_t)n + i);
        w_out[o] = expf(-expf(sum_slices(z, Sz, z_stride, o) + w0[i]));
    }
    if (t + 1 == cu_seqlens[seq + 1]) {
        float *kept = state + (size_t)slots[seq] * state_stride + state_off;
        for (int i = blockIdx.y * 256 + threadIdx.x; i < d; i += gridDim.y * 256) kept[i] = to_f32<T>(h[(size_t)t * d + i]);
    }
}

KESTREL_API int kestrel_time_mix_gates(const float *partial, int S, long long slice_stride, int ld, const float *z, int Sz, long long z_stride,
                                       const float *w0, float *r_out, float *k_out, float *v_out, float *w_out, int n, const void *h, int dtype, int d,
                                       float *state, long long state_stride, long long state_off, const int *seq_of_token, const int *cu_seqlens,
                                       const int *slots, int T, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && S > 0 && Sz > 0 && n > 0 && d > 0 && ld >= 3 * n && state_off >= 0, "time_mix_gates: bad sizes");
    const dim3 grid(T, T >= 256 ? 1 : (n + 255) / 256);
#define TG_GO(TT) kestrel_launch(time_mix_gates_kernel<TT>, grid, dim3(256), 0, stream, partial, S, (size_t)slice_stride, ld, z, Sz, (size_t)z_stride, w0, r_out, \
                                 k_out, v_out, w_out, n, (const TT *)h, d, state, (size_t)state_stride, (size_t)state_off, seq_of_token, cu_seqlens, slots)
    if (dtype == KESTREL_F32) TG_GO(float);
    else if (dtype == KESTREL_BF16) TG_GO(__nv_bfloat16);
    else return kestrel_fail(-2, "time_mix_gates: unknown dtype %d", dtype);
#undef TG_GO
    return kestrel_check_launch("time_mix_gates");
}

// ---- a step of few tokens: state, read-out, norm, gate of a (request, head); and the request's last h into its slot ------------
template <typename T, int VEC>
__global__ void __launch_bounds__(RST_THREADS)
time_mix_step_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, const float *__restrict__ z, int Sz, size_t z_stride,
                     const float *__restrict__ w0, const float *__restrict__ u, const float *__restrict__ norm_w, float eps, float scale,
                     const T *__restrict__ hrow, int width, float *__restrict__ state, size_t state_stride, size_t state_off, size_t last_off,
                     const int *__restrict__ cu_seqlens, const int *__restrict__ slots, T *__restrict__ out, long long ldo, int H, int d) {
    __shared__ float r_s[256], k_s[256], v_s[256], g_s[256], w_s[256], ru_s[256], part_s[RST_THREADS * VEC], red[RST_THREADS / 32];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, n = H * d;
    const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1];
    if (t0 == t1) return;
    float *slot = state + (size_t)slots[seq] * state_stride, *Sg = slot + state_off + (size_t)h * d * d;
    const RstLayout l = rst_layout<VEC>(d);
    for (int t = t0; t < t1; ++t) {
        const size_t row = (size_t)t * ld + (size_t)h * d;
        for (int i = tid; i < 4 * d; i += RST_THREADS) {
            const int what = i / d, c = i % d;
            const float x = sum_slices(p, S, slice_stride, row + (size_t)what * n + c);
            (what == 0 ? r_s : what == 1 ? k_s : what == 2 ? v_s : g_s)[c] = x;
        }
        for (int c = tid; c < d; c += RST_THREADS)
            w_s[c] = expf(-expf(sum_slices(z, Sz, z_stride, (size_t)t * n + (size_t)h * d + c) + w0[(size_t)h * d + c]));
        __syncthreads();
        float bonus = 0.f;                            // (r . (u k)) times v: the token's own write
        for (int c = tid; c < d; c += RST_THREADS) bonus = fmaf(r_s[c] * u[(size_t)h * d + c], k_s[c], bonus);
        bonus = rst_block_sum(bonus, red);
        if (l.rg < l.groups) {
            float acc[VEC], v[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) { acc[e] = 0.f; v[e] = v_s[l.c0 + e]; }
            for (int i0 = l.rg; i0 < d; i0 += 8 * l.groups) {          // eight rows' loads in flight
                float s[8][VEC];
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    const int i = i0 + r * l.groups;
                    if (i < d) rst_load<VEC>(s[r], Sg + (size_t)i * d + l.c0);
                }
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    const int i = i0 + r * l.groups;
                    if (i >= d) continue;
                    const float k = k_s[i], q = r_s[i], w = w_s[i];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        acc[e] = fmaf(s[r][e], q, acc[e]);
                        s[r][e] = fmaf(w, s[r][e], k * v[e]);
                    }
                    rst_store<VEC>(Sg + (size_t)i * d + l.c0, s[r]);
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) part_s[l.rg * d + l.c0 + e] = acc[e];
        }
        __syncthreads();
        float o = 0.f;
        if (tid < d) {                                // d <= RST_THREADS: a thread a value channel
            for (int r = 0; r < l.groups; ++r) o += part_s[r * d + tid];
            o = fmaf(bonus, v_s[tid], o);
        }
        const float tot = rst_block_sum(o * o, red);
        if (tid < d) {
            const float g = g_s[tid];
            out[(size_t)t * ldo + (size_t)h * d + tid] =
                from_f32<T>(o * (1.0f / sqrtf(tot / (float)d + eps)) * norm_w[(size_t)h * d + tid] * (g / (1.0f + expf(-g))) * scale);
        }
        __syncthreads();                              // the next token overwrites the shared rows
    }
    float *last = slot + last_off;                    // the heads share the row out
    for (int i = h * RST_THREADS + tid; i < width; i += H * RST_THREADS) last[i] = to_f32<T>(hrow[(size_t)(t1 - 1) * width + i]);
}

KESTREL_API int kestrel_time_mix_step(const float *partial, int S, long long slice_stride, int ld, const float *z, int Sz, long long z_stride, const float *w0,
                                      const float *u, const float *norm_w, float eps, float scale, const void *h, int width, float *state,
                                      long long state_stride, long long state_off, long long last_off, const int *cu_seqlens, const int *slots, void *out,
                                      long long ldo, int dtype, int nseq, int H, int d, cudaStream_t stream) {
    if (nseq == 0) return 0;
    KESTREL_REQUIRE(nseq > 0 && nseq <= 65535 && S > 0 && Sz > 0 && H > 0 && d > 0 && d <= 256 && ld >= 4 * H * d && width > 0 && state_off >= 0 &&
                    last_off >= state_off + (long long)H * d * d, "time_mix_step: bad sizes H=%d d=%d", H, d);
    const bool vec = d % 4 == 0 && state_stride % 4 == 0 && state_off % 4 == 0 && ((uintptr_t)state & 15) == 0;
#define TS_GO(TT, V) kestrel_launch(time_mix_step_kernel<TT, V>, dim3(H, nseq), dim3(RST_THREADS), 0, stream, partial, S, (size_t)slice_stride, ld, z, Sz, \
                                    (size_t)z_stride, w0, u, norm_w, eps, scale, (const TT *)h, width, state, (size_t)state_stride, (size_t)state_off, \
                                    (size_t)last_off, cu_seqlens, slots, (TT *)out, ldo, H, d)
    if (dtype == KESTREL_F32) { if (vec) TS_GO(float, 4); else TS_GO(float, 1); }
    else if (dtype == KESTREL_BF16) { if (vec) TS_GO(__nv_bfloat16, 4); else TS_GO(__nv_bfloat16, 1); }
    else return kestrel_fail(-2, "time_mix_step: unknown dtype %d", dtype);
#undef TS_GO
    return kestrel_check_launch("time_mix_step");
}
