// Short causal convolutions over time, one filter per channel, in front of recurrences and of attention:
//
//   y[t, c] = act( sum_j w[j, c] u[t - (taps - 1) + j, c] (+ b[c]) ),   act the identity or silu; w [taps][C]
//
// u are columns of a product (float32 slices); inputs before a request's first token of this step come from its state slot, which
// keeps the last taps - 1 of them (float32 [taps - 1][C], oldest first; zeros for a new request) and is brought up to date by a
// second kernel, after every reader of the old inputs is done.
#include "common.cuh"
#include <math.h>

#define SC_MAX_TAPS 9
#define SC_THREADS 128
#define SC_RUN 8          // tokens of a thread in steps of many

template <int VEC> __device__ __forceinline__ void sc_add(float (&x)[VEC], const float *__restrict__ p) {
    if constexpr (VEC == 1) {
        x[0] += p[0];
    } else {
        const float4 v = *reinterpret_cast<const float4 *>(p);
        x[0] += v.x; x[1] += v.y; x[2] += v.z; x[3] += v.w;
    }
}
template <int VEC> __device__ __forceinline__ void sc_store(float *dst, const float (&y)[VEC]) {
    if constexpr (VEC == 1) dst[0] = y[0];
    else *reinterpret_cast<float4 *>(dst) = make_float4(y[0], y[1], y[2], y[3]);
}
template <int VEC> __device__ __forceinline__ void sc_store(__nv_bfloat16 *dst, const float (&y)[VEC]) {
    if constexpr (VEC == 1) {
        dst[0] = __float2bfloat16_rn(y[0]);
    } else {
        __nv_bfloat162 a = __floats2bfloat162_rn(y[0], y[1]), b = __floats2bfloat162_rn(y[2], y[3]);
        *reinterpret_cast<uint2 *>(dst) = make_uint2(*reinterpret_cast<uint32_t *>(&a), *reinterpret_cast<uint32_t *>(&b));
    }
}

template <int N> struct ScCount { static constexpr int value = N; };

// A thread takes VEC neighbouring channels and RUN tokens, their inputs in registers.  TP >= taps: the filter is padded in front with
// zeros.
template <typename T, int VEC, int TP, int RUN>
__global__ void __launch_bounds__(SC_THREADS)
short_conv_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, int col0, const float *__restrict__ w, const float *__restrict__ b,
                  int taps, int silu, const float *__restrict__ state, size_t state_stride, size_t tail_off, const int *__restrict__ seq_of_token,
                  const int *__restrict__ cu_seqlens, const int *__restrict__ slots, T *__restrict__ out, int n_tokens, int C) {
    pdl_launch_dependents();
    const int c0 = (blockIdx.y * SC_THREADS + threadIdx.x) * VEC;
    if (c0 >= C) return;
    float f[TP][VEC], bias[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        bias[e] = b ? b[c0 + e] : 0.f;
#pragma unroll
        for (int j = 0; j < TP; ++j) f[j][e] = j >= TP - taps ? w[(size_t)(j - (TP - taps)) * C + c0 + e] : 0.f;
    }
    pdl_wait();
    const int t0 = blockIdx.x * RUN, t1 = min(t0 + RUN, n_tokens);
    // N tokens of one request from t on: all of their inputs and the filter's earlier ones in flight together
    auto go = [&](auto count, int t, int q) {
        constexpr int N = decltype(count)::value;
        const int first = cu_seqlens[q];
        const float *tail = state + (size_t)slots[q] * state_stride + tail_off;
        float x[TP - 1 + N][VEC];
#pragma unroll
        for (int j = 0; j < TP - 1 + N; ++j) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) x[j][e] = 0.f;
        }
        const int n0 = t - first - (TP - 1);                  // the first input, among this step's tokens of the request
        const float *src = p + (size_t)t * ld + col0 + c0 - (size_t)(TP - 1) * ld;
        for (int s = 0; s < S; ++s, src += slice_stride) {
#pragma unroll
            for (int j = 0; j < TP - 1 + N; ++j)
                if (j >= TP - taps && n0 + j >= 0 && t + j - (TP - 1) < t1) sc_add<VEC>(x[j], src + (size_t)j * ld);
        }
        if (n0 < 0) {
#pragma unroll
            for (int j = 0; j < TP - 1; ++j)
                if (j >= TP - taps && n0 + j < 0) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) x[j][e] = tail[(size_t)(taps - 1 + n0 + j) * C + c0 + e];
                }
        }
#pragma unroll
        for (int k = 0; k < N; ++k) {
            if (t + k >= t1) break;
            float y[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                float a = 0.f;
#pragma unroll
                for (int j = 0; j < TP; ++j) a = fmaf(f[j][e], x[k + j][e], a);
                a += bias[e];
                y[e] = !silu ? a : sizeof(T) == 2 ? __fdividef(a, 1.0f + __expf(-a)) : a / (1.0f + expf(-a));
            }
            sc_store<VEC>(out + (size_t)(t + k) * C + c0, y);
        }
    };
    const int q0 = seq_of_token[t0];
    if (RUN > 1 && seq_of_token[t1 - 1] == q0) {
        go(ScCount<RUN>(), t0, q0);
    } else {
        for (int t = t0; t < t1; ++t) go(ScCount<1>(), t, seq_of_token[t]);
    }
}

__global__ void short_conv_tail_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, int col0, int taps, float *__restrict__ state,
                                       size_t state_stride, size_t tail_off, const int *__restrict__ cu_seqlens, const int *__restrict__ slots, int C) {
    pdl_launch_dependents();
    pdl_wait();
    const int seq = blockIdx.x, first = cu_seqlens[seq], n_tok = cu_seqlens[seq + 1] - first;
    if (n_tok == 0) return;
    float *tail = state + (size_t)slots[seq] * state_stride + tail_off;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
        float keep[SC_MAX_TAPS - 1];
#pragma unroll
        for (int r = 0; r < SC_MAX_TAPS - 1; ++r)
            if (r < taps - 1) {
                const int n = n_tok - (taps - 1) + r;
                keep[r] = n >= 0 ? sum_slices(p, S, slice_stride, (size_t)(first + n) * ld + col0 + c) : tail[(size_t)(taps - 1 + n) * C + c];
            }
#pragma unroll
        for (int r = 0; r < SC_MAX_TAPS - 1; ++r)
            if (r < taps - 1) tail[(size_t)r * C + c] = keep[r];
    }
}

template <typename T, int VEC>
static void sc_launch(const float *p, int S, size_t ss, int ld, int col0, const float *w, const float *b, int taps, int silu, const float *state, size_t st,
                      size_t to, const int *seq_of_token, const int *cu, const int *slots, T *out, int n_tokens, int C, cudaStream_t stream) {
    const int run = n_tokens >= 512 ? SC_RUN : 1;
    const dim3 grid((n_tokens + run - 1) / run, (C / VEC + SC_THREADS - 1) / SC_THREADS);
#define SC_GO(TP) if (run > 1) SC_RUN_GO(TP, SC_RUN); else SC_RUN_GO(TP, 1)
#define SC_RUN_GO(TP, R) kestrel_launch(short_conv_kernel<T, VEC, TP, R>, grid, dim3(SC_THREADS), 0, stream, p, S, ss, ld, col0, w, b, taps, silu, state, st, to, \
                                 seq_of_token, cu, slots, out, n_tokens, C)
    if (taps <= 2) { SC_GO(2); }
    else if (taps <= 4) { SC_GO(4); }
    else { SC_GO(SC_MAX_TAPS); }
#undef SC_RUN_GO
#undef SC_GO
}

KESTREL_API int kestrel_short_conv_tail(const float *partial, int S, long long slice_stride, int ld, int col0, int taps, float *state, long long state_stride,
                                        long long tail_off, const int *cu_seqlens, const int *slots, int nseq, int C, cudaStream_t stream) {
    if (nseq == 0 || taps == 1) return 0;
    KESTREL_REQUIRE(nseq > 0 && C > 0 && S > 0 && col0 >= 0 && col0 + C <= ld && taps >= 1 && taps <= SC_MAX_TAPS, "short_conv_tail: bad sizes (taps %d)", taps);
    kestrel_launch(short_conv_tail_kernel, dim3(nseq, (C + 255) / 256), dim3(256), 0, stream, partial, S, (size_t)slice_stride, ld, col0, taps, state,
                   (size_t)state_stride, (size_t)tail_off, cu_seqlens, slots, C);
    return kestrel_check_launch("short_conv_tail");
}

KESTREL_API int kestrel_short_conv(const float *partial, int S, long long slice_stride, int ld, int col0, const float *w, const float *bias, int taps,
                                   int silu, float *state, long long state_stride, long long tail_off, const int *seq_of_token, const int *cu_seqlens,
                                   const int *slots, void *out, int dtype, int T, int nseq, int C, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && nseq > 0 && C > 0 && S > 0 && col0 >= 0 && col0 + C <= ld && taps >= 1 && taps <= SC_MAX_TAPS, "short_conv: bad sizes (taps %d)", taps);
    KESTREL_REQUIRE(dtype == KESTREL_F32 || dtype == KESTREL_BF16, "short_conv: unknown dtype %d", dtype);
    const bool vec = C % 4 == 0 && ld % 4 == 0 && col0 % 4 == 0 && slice_stride % 4 == 0 && (((uintptr_t)partial | (uintptr_t)out) & 15) == 0;
#define SC_ARGS(TT) partial, S, (size_t)slice_stride, ld, col0, w, bias, taps, silu, (const float *)state, (size_t)state_stride, (size_t)tail_off, seq_of_token, \
                    cu_seqlens, slots, (TT *)out, T, C, stream
    if (dtype == KESTREL_F32) { if (vec) sc_launch<float, 4>(SC_ARGS(float)); else sc_launch<float, 1>(SC_ARGS(float)); }
    else { if (vec) sc_launch<__nv_bfloat16, 4>(SC_ARGS(__nv_bfloat16)); else sc_launch<__nv_bfloat16, 1>(SC_ARGS(__nv_bfloat16)); }
#undef SC_ARGS
    int rc = kestrel_check_launch("short_conv");
    if (rc) return rc;
    return kestrel_short_conv_tail(partial, S, slice_stride, ld, col0, taps, state, state_stride, tail_off, cu_seqlens, slots, nseq, C, stream);
}
