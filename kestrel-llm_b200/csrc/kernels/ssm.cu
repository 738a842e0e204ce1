// A state-space mixer with a scalar decay per head (Mamba-2).  Per head n, with B and C of its group and a step size dt:
//
//     S_t = exp(-exp(A_log) dt_t) S_{t-1} + dt_t B_t x_t^T,    y_t = S_t^T C_t + D x_t
//
// x | B | C come out of a short convolution (short_conv.cu) as columns of `act`; dt = softplus(logit + dt_bias), float32.  y is
// multiplied by silu(z) and normed in equal parts of the concatenated heads, after the gate.
//
// Steps of few tokens: `step` does everything between the input product and the norm.  Prompt portions in bfloat16: `steps` and
// decay_chunks.cu.  Both leave the gated y for `part_norm`.  float32 and what lies between:
//   expand        what the sequential scan of linear_recurrence.cu takes, head by head: r = C, k = B, v = dt x, w = the decay
//   out           + D x, gate, norm per part, weight, to the storage type
#include "common.cuh"
#include "recurrence_step.cuh"
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

// ---- step sizes and logarithms of the decays, for the chunked form (decay_chunks.cu) -----------------------------------------
__global__ void __launch_bounds__(128)
ssm_steps_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, int col_dt, const float *__restrict__ dt_bias,
                 const float *__restrict__ A_log, float *__restrict__ step, float *__restrict__ log_decay, int H, size_t total) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t idx = (size_t)blockIdx.x * 128 + threadIdx.x;
    if (idx >= total) return;
    const size_t t = idx / H;
    const int h = (int)(idx % H);
    const float dt = ssm_softplus(sum_slices(p, S, slice_stride, t * ld + col_dt + h) + dt_bias[h]);
    step[idx] = dt;
    log_decay[idx] = -expf(A_log[h]) * dt;
}

KESTREL_API int kestrel_ssm_steps(const float *partial, int S, long long slice_stride, int ld, int col_dt, const float *dt_bias, const float *A_log,
                                  float *step, float *log_decay, int T, int H, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && S > 0 && H > 0 && col_dt >= 0 && col_dt + H <= ld, "ssm_steps: bad sizes");
    const size_t total = (size_t)T * H;
    kestrel_launch(ssm_steps_kernel, dim3((unsigned)((total + 127) / 128)), dim3(128), 0, stream, partial, S, (size_t)slice_stride, ld, col_dt, dt_bias, A_log,
                   step, log_decay, H, total);
    return kestrel_check_launch("ssm_steps");
}

// ---- a step of few tokens: convolution, state, read-out, skip and gate of a (request, head); y [T, H P] float32 ----------------
template <int VEC>
__global__ void __launch_bounds__(RST_THREADS)
ssm_step_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, int col_z, int col_x, int col_dt, const float *__restrict__ conv_w,
                const float *__restrict__ conv_b, int taps, const float *__restrict__ dt_bias, const float *__restrict__ A_log, const float *__restrict__ D,
                float *__restrict__ state, size_t state_stride, size_t tail_off, const int *__restrict__ cu_seqlens, const int *__restrict__ slots,
                float *__restrict__ y, int H, int G, int N, int P) {
    __shared__ float x_s[256], b_s[256], c_s[256], z_s[256], part_s[RST_THREADS * VEC], sc[2];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, g = h / (H / G), inner = H * P, C = inner + 2 * G * N;
    const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1];
    if (t0 == t1) return;
    float *slot = state + (size_t)slots[seq] * state_stride, *Sg = slot + (size_t)h * N * P;
    const float *tail = slot + tail_off;
    const RstLayout l = rst_layout<VEC>(P);
    for (int t = t0; t < t1; ++t) {
        for (int u = tid; u < 2 * P + 2 * N + 1; u += RST_THREADS) {
            if (u < P + 2 * N) {
                const int c = u < P ? h * P + u : (u < P + N ? inner + g * N + u - P : inner + G * N + g * N + u - P - N);
                const float a = rst_conv(p, S, slice_stride, ld, col_x + c, conv_w, taps, tail, C, c, t0, t) + conv_b[c];
                const float v = a / (1.0f + expf(-a));
                if (u < P) x_s[u] = v;
                else if (u < P + N) b_s[u - P] = v;
                else c_s[u - P - N] = v;
            } else if (u < 2 * P + 2 * N) {
                const int i = u - P - 2 * N;
                const float z = sum_slices(p, S, slice_stride, (size_t)t * ld + col_z + h * P + i);
                z_s[i] = z / (1.0f + expf(-z));
            } else {
                const float dt = ssm_softplus(sum_slices(p, S, slice_stride, (size_t)t * ld + col_dt + h) + dt_bias[h]);
                sc[0] = dt;
                sc[1] = expf(-expf(A_log[h]) * dt);
            }
        }
        __syncthreads();
        if (l.rg < l.groups) {
            const float dec = sc[1], dt = sc[0];
            float acc[VEC], v[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) { acc[e] = 0.f; v[e] = dt * x_s[l.c0 + e]; }
            for (int i0 = l.rg; i0 < N; i0 += 8 * l.groups) {          // eight rows' loads in flight
                float s[8][VEC];
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    const int i = i0 + r * l.groups;
                    if (i < N) rst_load<VEC>(s[r], Sg + (size_t)i * P + l.c0);
                }
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    const int i = i0 + r * l.groups;
                    if (i >= N) continue;
                    const float b = b_s[i], c = c_s[i];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        s[r][e] = fmaf(dec, s[r][e], b * v[e]);
                        acc[e] = fmaf(s[r][e], c, acc[e]);
                    }
                    rst_store<VEC>(Sg + (size_t)i * P + l.c0, s[r]);
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) part_s[l.rg * P + l.c0 + e] = acc[e];
        }
        __syncthreads();
        if (tid < P) {                                // P <= RST_THREADS: a thread a value channel
            float o = 0.f;
            for (int r = 0; r < l.groups; ++r) o += part_s[r * P + tid];
            y[(size_t)t * inner + h * P + tid] = fmaf(D[h], x_s[tid], o) * z_s[tid];
        }
        __syncthreads();                              // the next token overwrites the shared rows; a thread's state rows are its own
    }
}

KESTREL_API int kestrel_ssm_step(const float *partial, int S, long long slice_stride, int ld, int col_z, int col_x, int col_dt, const float *conv_w,
                                 const float *conv_b, int taps, const float *dt_bias, const float *A_log, const float *D, float *state,
                                 long long state_stride, long long tail_off, const int *cu_seqlens, const int *slots, float *y, int nseq, int H, int G, int N,
                                 int P, cudaStream_t stream) {
    if (nseq == 0) return 0;
    KESTREL_REQUIRE(nseq > 0 && nseq <= 65535 && S > 0 && H > 0 && G > 0 && H % G == 0 && N > 0 && N <= 256 && P > 0 && P <= 256 && taps >= 1 && taps <= 9 &&
                    tail_off >= (long long)H * N * P, "ssm_step: bad sizes H=%d N=%d P=%d", H, N, P);
    const bool vec = P % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
#define SS_GO(V) kestrel_launch(ssm_step_kernel<V>, dim3(H, nseq), dim3(RST_THREADS), 0, stream, partial, S, (size_t)slice_stride, ld, col_z, col_x, col_dt, conv_w, \
                                conv_b, taps, dt_bias, A_log, D, state, (size_t)state_stride, (size_t)tail_off, cu_seqlens, slots, y, H, G, N, P)
    if (vec) SS_GO(4);
    else SS_GO(1);
#undef SS_GO
    int rc = kestrel_check_launch("ssm_step");
    if (rc) return rc;
    return kestrel_short_conv_tail(partial, S, slice_stride, ld, col_x, taps, state, state_stride, tail_off, cu_seqlens, slots, nseq, H * P + 2 * G * N, stream);
}

// ---- rows normed in equal parts: out = y / sqrt(mean(y^2) + eps) per part * w -------------------------------------------------
template <typename T, int VEC>
__global__ void __launch_bounds__(512)
part_norm_kernel(const float *__restrict__ y, const float *__restrict__ w, float eps, T *__restrict__ out, int inner, int n) {
    __shared__ float red[16];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, c0 = blockIdx.y * n, nt = blockDim.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float *src = y + (size_t)t * inner + c0;
    T *dst = out + (size_t)t * inner + c0;
    float v[4][VEC], ss = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {                     // the first four of a thread's places in registers, the rest read again
        const int i = (threadIdx.x + k * nt) * VEC;
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[k][e] = 0.f;
        if (i < n) rst_load<VEC>(v[k], src + i);
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(v[k][e], v[k][e], ss);
    }
    for (int i = (threadIdx.x + 4 * nt) * VEC; i < n; i += nt * VEC) {
        float x[VEC];
        rst_load<VEC>(x, src + i);
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(x[e], x[e], ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int k = 0; k < nt / 32; ++k) tot += red[k];
    const float mul = 1.0f / sqrtf(tot / (float)n + eps);
    auto put = [&](int i, const float (&x)[VEC]) {
        if constexpr (VEC == 4 && sizeof(T) == 2) {
            __nv_bfloat162 a = __floats2bfloat162_rn(x[0] * mul * w[c0 + i], x[1] * mul * w[c0 + i + 1]);
            __nv_bfloat162 b = __floats2bfloat162_rn(x[2] * mul * w[c0 + i + 2], x[3] * mul * w[c0 + i + 3]);
            *reinterpret_cast<uint2 *>(dst + i) = make_uint2(*reinterpret_cast<uint32_t *>(&a), *reinterpret_cast<uint32_t *>(&b));
        } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) dst[i + e] = from_f32<T>(x[e] * mul * w[c0 + i + e]);
        }
    };
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const int i = (threadIdx.x + k * nt) * VEC;
        if (i < n) put(i, v[k]);
    }
    for (int i = (threadIdx.x + 4 * nt) * VEC; i < n; i += nt * VEC) {
        float x[VEC];
        rst_load<VEC>(x, src + i);
        put(i, x);
    }
}

KESTREL_API int kestrel_part_norm(const float *y, const float *w, float eps, void *out, int dtype, int T, int inner, int parts, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && inner > 0 && parts > 0 && inner % parts == 0 && parts <= 65535, "part_norm: bad sizes");
    const int n = inner / parts, vec = n % 4 == 0 && (((uintptr_t)y | (uintptr_t)out) & 15) == 0 ? 4 : 1;
    int nt = ((n + vec - 1) / vec + 31) / 32 * 32;
    if (nt > 512) nt = 512;
#define PN_GO(TT, V) kestrel_launch(part_norm_kernel<TT, V>, dim3(T, parts), dim3(nt), 0, stream, y, w, eps, (TT *)out, inner, n)
    if (dtype == KESTREL_F32) { if (vec == 4) PN_GO(float, 4); else PN_GO(float, 1); }
    else if (dtype == KESTREL_BF16) { if (vec == 4) PN_GO(__nv_bfloat16, 4); else PN_GO(__nv_bfloat16, 1); }
    else return kestrel_fail(-2, "part_norm: unknown dtype %d", dtype);
#undef PN_GO
    return kestrel_check_launch("part_norm");
}
