// A recurrent mixer: the gated delta rule with one decay per key channel, or one per head.  Per head, with a state S [d, dv] that starts at zero and is
// carried from token to token of a request (float32, in the request's state slot):
//
//     S <- diag(a_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
//
// The read-out sees the token's own write.  Everything that enters the recurrence is float32.
//
// Kernels, in the order of a step:
//   (short_conv.cu) q, k, v out of the fused product through a causal convolution and silu
//   gates         q, k made unit vectors per head (x / sqrt(sum x^2 + 1e-6)), q scaled by d^-1/2;
//                 beta = sigmoid(.); a = exp(-exp(A_log[h]) softplus(. + dt_bias)),
//                 the dot a column per key channel, or one per head that all of its channels take
//   scan          the recurrence; a value column of S stays in the registers of eight lanes (an
//                 eighth of the key channels each), so S^T k and S^T q are sums inside a thread
//                 and one fixed shuffle tree - a token's result does not depend on how the
//                 request was cut into steps or on the batch
//   out_norm_gate o / sqrt(mean(o^2) + eps) * w * sigmoid(gate) per head, in the storage type
#include "common.cuh"
#include "recurrence_step.cuh"
#include <math.h>

// sum of a product's slices at (token, column)
__device__ __forceinline__ float slices_at(const float *p, int S, size_t slice_stride, size_t off) {
    return sum_slices(p, S, slice_stride, off);
}

// act [T, C] = q (G*d) | k (G*d) | v (H*dv) after convolution and silu
__global__ void __launch_bounds__(128)
delta_gates_kernel(const float *__restrict__ act, int C, const float *__restrict__ partial, int S, size_t slice_stride, int ld, int col_beta,
                   const float *__restrict__ a_part, int Sa, size_t a_stride, int a_ld, int col_a, int per_head, const float *__restrict__ A_log,
                   const float *__restrict__ dt_bias, float *__restrict__ qn, float *__restrict__ kn, float *__restrict__ decay,
                   float *__restrict__ beta, int H, int G, int d) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float q_scale = 1.0f / sqrtf((float)d);
    for (int r = warp; r < 2 * G; r += 4) {                // q heads, then k heads
        const float *x = act + (size_t)t * C + (size_t)r * d;
        float ss = 0.f;
        for (int i = lane; i < d; i += 32) ss = fmaf(x[i], x[i], ss);
        ss = warp_sum(ss);
        const float mul = (1.0f / sqrtf(ss + 1e-6f)) * (r < G ? q_scale : 1.0f);
        float *dst = r < G ? qn + ((size_t)t * G + r) * d : kn + ((size_t)t * G + (r - G)) * d;
        for (int i = lane; i < d; i += 32) dst[i] = x[i] * mul;
    }
    for (int idx = threadIdx.x; idx < H * d; idx += 128) {
        const int h = idx / d;
        const int c = per_head ? h : idx;
        const float a = slices_at(a_part, Sa, a_stride, (size_t)t * a_ld + col_a + c) + dt_bias[c];
        const float sp = a > 20.f ? a : log1pf(expf(a));
        decay[(size_t)t * H * d + idx] = expf(-expf(A_log[h]) * sp);
    }
    for (int h = threadIdx.x; h < H; h += 128) {
        const float z = slices_at(partial, S, slice_stride, (size_t)t * ld + col_beta + h);
        beta[(size_t)t * H + h] = 1.0f / (1.0f + expf(-z));
    }
}

#define DR_TC 8        // tokens staged in shared memory at a time
#define DR_LPC 8       // lanes that share a value column's key channels
#define DR_COLS (128 / DR_LPC)      // value columns of a CTA of four warps

__device__ __forceinline__ void dr_cp_async(float *dst, const float *src, bool vec4) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    if (vec4) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

// A CTA of four warps takes DR_COLS value columns of one (request, head); the DR_LPC lanes of a
// column hold interleaved parts of its D (padded) key channels: lane part s owns channels
// 4 (DR_LPC m + s) + {0..3}.  Per token a thread does D / DR_LPC decays and multiply-adds twice
// (S^T k, then the write and S^T q) on four partial sums each, and the lanes of a column add their
// parts in a fixed shuffle tree.  The time of a token is the latency of this chain, so the parts
// are short: with four lanes a column a token took 0.41 us, with eight it takes less.  k, q, the decays, v and beta of DR_TC tokens are staged in
// shared memory with cp.async, the next stage in flight while the current one is used.
template <int D>
__global__ void __launch_bounds__(128)
delta_scan_kernel(const float *__restrict__ qn, const float *__restrict__ kn, const float *__restrict__ decay,
                  const float *__restrict__ act, int C, int col_v, const float *__restrict__ beta, float *__restrict__ state,
                  size_t state_stride, const int *__restrict__ cu_seqlens, const int *__restrict__ slots,
                  float *__restrict__ out, int H, int G, int d, int dv) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int STAGE = DR_TC * (3 * D + 32) + DR_TC;      // floats: k, q, a [TC][D]; v [TC][32, DR_COLS used]; beta [TC]
    constexpr int M = D / (4 * DR_LPC);                      // float4s of a thread's part
    extern __shared__ float4 dr_smem4[];
    float *sm = reinterpret_cast<float *>(dr_smem4);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int part = lane % DR_LPC, cj = lane / DR_LPC;
    const int jl = warp * (32 / DR_LPC) + cj, j = blockIdx.x * DR_COLS + jl, h = blockIdx.y, seq = blockIdx.z;
    const int g = h / (H / G);
    const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1];
    const bool live = j < dv;
    const bool vec4 = d % 4 == 0;
    float *Sg = state + (size_t)slots[seq] * state_stride + (size_t)h * d * dv;     // [d][dv]
    float Sc[M][4];
#pragma unroll
    for (int m = 0; m < M; ++m)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int i = 4 * (DR_LPC * m + part) + c;
            Sc[m][c] = (i < d && live) ? Sg[(size_t)i * dv + j] : 0.f;
        }
    for (int idx = tid; idx < 2 * STAGE; idx += 128) sm[idx] = 0.f;       // the padded channels stay zero
    __syncthreads();

    auto issue = [&](int tb, int stage) {
        float *sk = sm + (size_t)stage * STAGE, *sq = sk + DR_TC * D, *sa = sq + DR_TC * D, *sv = sa + DR_TC * D, *sb = sv + DR_TC * 32;
        const int per = vec4 ? d / 4 : d, w = vec4 ? 4 : 1;
        for (int idx = tid; idx < DR_TC * per; idx += 128) {
            const int c = idx / per, e = (idx % per) * w, t = tb + c;
            if (t < t1) {
                dr_cp_async(sk + c * D + e, kn + ((size_t)t * G + g) * d + e, vec4);
                dr_cp_async(sq + c * D + e, qn + ((size_t)t * G + g) * d + e, vec4);
                dr_cp_async(sa + c * D + e, decay + ((size_t)t * H + h) * d + e, vec4);
            }
        }
        for (int idx = tid; idx < DR_TC * 32; idx += 128) {
            const int c = idx / 32, jj = idx % 32, t = tb + c, col = blockIdx.x * DR_COLS + jj;
            if (t < t1 && jj < DR_COLS && col < dv) dr_cp_async(sv + c * 32 + jj, act + (size_t)t * C + col_v + (size_t)h * dv + col, false);
        }
        if (tid < DR_TC && tb + tid < t1) dr_cp_async(sb + tid, beta + (size_t)(tb + tid) * H + h, false);
    };
    if (t0 < t1) issue(t0, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    int stage = 0;
    for (int tb = t0; tb < t1; tb += DR_TC, stage ^= 1) {
        if (tb + DR_TC < t1) issue(tb + DR_TC, stage ^ 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const float *sk = sm + (size_t)stage * STAGE, *sq = sk + DR_TC * D, *sa = sq + DR_TC * D, *sv = sa + DR_TC * D, *sb = sv + DR_TC * 32;
        const int n = min(DR_TC, t1 - tb);
#pragma unroll
        for (int c = 0; c < DR_TC; ++c) {             // unrolled: the next token's operands are fetched under this token's chain
            if (c >= n) break;
            const float4 *k4 = reinterpret_cast<const float4 *>(sk + c * D), *q4 = reinterpret_cast<const float4 *>(sq + c * D),
                         *a4 = reinterpret_cast<const float4 *>(sa + c * D);
            float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
            for (int m = 0; m < M; ++m) {
                const float4 kk = k4[DR_LPC * m + part], aa = a4[DR_LPC * m + part];
                Sc[m][0] *= aa.x; s0 = fmaf(Sc[m][0], kk.x, s0);
                Sc[m][1] *= aa.y; s1 = fmaf(Sc[m][1], kk.y, s1);
                Sc[m][2] *= aa.z; s2 = fmaf(Sc[m][2], kk.z, s2);
                Sc[m][3] *= aa.w; s3 = fmaf(Sc[m][3], kk.w, s3);
            }
            float acc = (s0 + s1) + (s2 + s3);
#pragma unroll
            for (int sh = 1; sh < DR_LPC; sh <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, sh);
            const float u = sb[c] * (sv[c * 32 + jl] - acc);
            s0 = s1 = s2 = s3 = 0.f;
#pragma unroll
            for (int m = 0; m < M; ++m) {
                const float4 kk = k4[DR_LPC * m + part], qq = q4[DR_LPC * m + part];
                Sc[m][0] = fmaf(kk.x, u, Sc[m][0]); s0 = fmaf(Sc[m][0], qq.x, s0);
                Sc[m][1] = fmaf(kk.y, u, Sc[m][1]); s1 = fmaf(Sc[m][1], qq.y, s1);
                Sc[m][2] = fmaf(kk.z, u, Sc[m][2]); s2 = fmaf(Sc[m][2], qq.z, s2);
                Sc[m][3] = fmaf(kk.w, u, Sc[m][3]); s3 = fmaf(Sc[m][3], qq.w, s3);
            }
            float o = (s0 + s1) + (s2 + s3);
#pragma unroll
            for (int sh = 1; sh < DR_LPC; sh <<= 1) o += __shfl_xor_sync(0xffffffffu, o, sh);
            if (live && part == 0) out[((size_t)(tb + c) * H + h) * dv + j] = o;
        }
        __syncthreads();                              // the stage may be filled again
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (live) {
#pragma unroll
        for (int m = 0; m < M; ++m)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int i = 4 * (DR_LPC * m + part) + c;
                if (i < d) Sg[(size_t)i * dv + j] = Sc[m][c];
            }
    }
}

template <typename T>
__global__ void __launch_bounds__(128)
delta_out_kernel(const float *__restrict__ o, const float *__restrict__ w, float eps, const float *__restrict__ g_part, int Sg,
                 size_t g_stride, T *__restrict__ out, int H, int dv) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int h = warp; h < H; h += 4) {
        const size_t base = ((size_t)t * H + h) * dv;
        float ss = 0.f;
        for (int i = lane; i < dv; i += 32) ss = fmaf(o[base + i], o[base + i], ss);
        ss = warp_sum(ss);
        const float r = 1.0f / sqrtf(ss / (float)dv + eps);
        for (int i = lane; i < dv; i += 32) {
            const float z = slices_at(g_part, Sg, g_stride, base + i);
            out[base + i] = from_f32<T>(o[base + i] * r * w[i] * (1.0f / (1.0f + expf(-z))));
        }
    }
}

KESTREL_API int kestrel_delta_gates(const float *act, int C, const float *partial, int S, long long slice_stride, int ld, int col_beta,
                                    const float *a_part, int Sa, long long a_stride, int a_ld, int col_a, int per_head, const float *A_log,
                                    const float *dt_bias, float *qn, float *kn, float *decay, float *beta, int T, int H, int G, int d, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && H > 0 && G > 0 && H % G == 0 && d > 0 && Sa > 0 && col_a >= 0 && col_a + (per_head ? H : H * d) <= a_ld, "delta_gates: bad sizes");
    kestrel_launch(delta_gates_kernel, dim3(T), dim3(128), 0, stream, act, C, partial, S, (size_t)slice_stride, ld, col_beta, a_part, Sa,
                   (size_t)a_stride, a_ld, col_a, per_head, A_log, dt_bias, qn, kn, decay, beta, H, G, d);
    return kestrel_check_launch("delta_gates");
}

KESTREL_API int kestrel_delta_scan(const float *qn, const float *kn, const float *decay, const float *act, int C, int col_v, const float *beta,
                                   float *state, long long state_stride, const int *cu_seqlens, const int *slots, float *out, int nseq,
                                   int H, int G, int d, int dv, cudaStream_t stream) {
    if (nseq == 0) return 0;
    KESTREL_REQUIRE(nseq > 0 && H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0, "delta_scan: bad sizes");
    KESTREL_REQUIRE(d <= 256, "delta_scan: key size %d exceeds 256", d);
    KESTREL_REQUIRE(H <= 65535 && nseq <= 65535, "delta_scan: grid too large");
    dim3 grid((dv + DR_COLS - 1) / DR_COLS, H, nseq);
#define DR_LAUNCH(D)                                                                                                                  \
    {                                                                                                                                 \
        static bool attr_set = false;                                                                                                 \
        if (!attr_set && cudaFuncSetAttribute(delta_scan_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize,                      \
                                              KESTREL_SMEM_MAX_DYNAMIC) != cudaSuccess)                                               \
            return kestrel_fail(-3, "delta_scan: cannot set the shared memory size");                                                 \
        attr_set = true;                                                                                                              \
    }                                                                                                                                 \
    kestrel_launch(delta_scan_kernel<D>, grid, dim3(128),                                                                             \
                   kestrel_spread_smem((long)grid.x * grid.y * grid.z, (size_t)2 * (DR_TC * (3 * D + 32) + DR_TC) * sizeof(float)),   \
                   stream, qn, kn, decay, act, C, col_v, beta, state, (size_t)state_stride, cu_seqlens, slots, out, H, G, d, dv)
    if (d <= 32) { DR_LAUNCH(32); }
    else if (d <= 64) { DR_LAUNCH(64); }
    else if (d <= 128) { DR_LAUNCH(128); }
    else { DR_LAUNCH(256); }
#undef DR_LAUNCH
    return kestrel_check_launch("delta_scan");
}

KESTREL_API int kestrel_delta_out(const float *o, const float *w, float eps, const float *g_part, int Sg, long long g_stride, void *out,
                                  int dtype, int T, int H, int dv, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && H > 0 && dv > 0 && Sg > 0, "delta_out: bad sizes");
    if (dtype == KESTREL_F32)
        kestrel_launch(delta_out_kernel<float>, dim3(T), dim3(128), 0, stream, o, w, eps, g_part, Sg, (size_t)g_stride, (float *)out, H, dv);
    else if (dtype == KESTREL_BF16)
        kestrel_launch(delta_out_kernel<__nv_bfloat16>, dim3(T), dim3(128), 0, stream, o, w, eps, g_part, Sg, (size_t)g_stride, (__nv_bfloat16 *)out, H, dv);
    else
        return kestrel_fail(-2, "delta_out: unknown dtype %d", dtype);
    return kestrel_check_launch("delta_out");
}

// ---- one decay per head, a step of few tokens: everything between the fused product and the output product --------------------
// columns [q: G d | k: G d | v: H dv] through the convolution, gate logits at col_g, beta and decay logits a head at col_beta, col_a
template <typename T, int VEC, int ROWS>
__global__ void __launch_bounds__(RST_THREADS)
delta_head_step_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, int col_g, int col_beta, int col_a, const float *__restrict__ conv_w,
                       int taps, const float *__restrict__ A_log, const float *__restrict__ dt_bias, const float *__restrict__ norm_w, float eps,
                       float *__restrict__ state, size_t state_stride, size_t tail_off, const int *__restrict__ cu_seqlens, const int *__restrict__ slots,
                       T *__restrict__ out, int H, int G, int d, int dv) {
    __shared__ float q_s[256], k_s[256], v_s[256], g_s[256], u_s[256], part_s[RST_THREADS * VEC], red[RST_THREADS / 32], sc[4];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, hk = h / (H / G), C = 2 * G * d + H * dv;
    const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1];
    if (t0 == t1) return;
    float *slot = state + (size_t)slots[seq] * state_stride, *Sg = slot + (size_t)h * d * dv;
    const float *tail = slot + tail_off;
    const RstLayout l = rst_layout<VEC>(dv);
    float s[ROWS][VEC];
    const bool mine = l.rg < l.groups;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const int i = l.rg + r * l.groups;
#pragma unroll
        for (int e = 0; e < VEC; ++e) s[r][e] = 0.f;
        if (mine && i < d) rst_load<VEC>(s[r], Sg + (size_t)i * dv + l.c0);
    }
    for (int t = t0; t < t1; ++t) {
        for (int u = tid; u < 2 * d + 2 * dv + 2; u += RST_THREADS) {
            if (u < 2 * d + dv) {
                const int c = u < d ? hk * d + u : (u < 2 * d ? (G + hk) * d + u - d : 2 * G * d + h * dv + u - 2 * d);
                const float a = rst_conv(p, S, slice_stride, ld, c, conv_w, taps, tail, C, c, t0, t), y = a / (1.0f + expf(-a));
                if (u < d) q_s[u] = y;
                else if (u < 2 * d) k_s[u - d] = y;
                else v_s[u - 2 * d] = y;
            } else if (u < 2 * d + 2 * dv) {
                const int i = u - 2 * d - dv;
                g_s[i] = sum_slices(p, S, slice_stride, (size_t)t * ld + col_g + h * dv + i);
            } else if (u == 2 * d + 2 * dv) {
                sc[0] = 1.0f / (1.0f + expf(-sum_slices(p, S, slice_stride, (size_t)t * ld + col_beta + h)));
            } else {
                const float a = sum_slices(p, S, slice_stride, (size_t)t * ld + col_a + h) + dt_bias[h];
                sc[1] = expf(-expf(A_log[h]) * (a > 20.f ? a : log1pf(expf(a))));
            }
        }
        __syncthreads();
        if (warp < 2) {                               // q's and k's unit factors
            const float *x = warp == 0 ? q_s : k_s;
            float ss = 0.f;
            for (int i = lane; i < d; i += 32) ss = fmaf(x[i], x[i], ss);
            ss = warp_sum(ss);
            if (lane == 0) sc[2 + warp] = (1.0f / sqrtf(ss + 1e-6f)) * (warp == 0 ? 1.0f / sqrtf((float)d) : 1.0f);
        }
        __syncthreads();
        const float beta = sc[0], dec = sc[1], qf = sc[2], kf = sc[3];
        float acc[VEC];
        if (mine) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
#pragma unroll
            for (int r = 0; r < ROWS; ++r) {
                const int i = l.rg + r * l.groups;
                const float k = i < d ? k_s[i] : 0.f;
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[r][e] *= dec;
                    acc[e] = fmaf(s[r][e], k, acc[e]);
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) part_s[l.rg * dv + l.c0 + e] = acc[e];
        }
        __syncthreads();
        if (tid < dv) {                               // dv <= RST_THREADS: a thread a value channel
            float held = 0.f;
            for (int r = 0; r < l.groups; ++r) held += part_s[r * dv + tid];
            u_s[tid] = beta * (v_s[tid] - held * kf) * kf;      // times k's factor: the write is k_s * this
        }
        __syncthreads();
        if (mine) {
            float u[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) { acc[e] = 0.f; u[e] = u_s[l.c0 + e]; }
#pragma unroll
            for (int r = 0; r < ROWS; ++r) {
                const int i = l.rg + r * l.groups;
                const float k = i < d ? k_s[i] : 0.f, q = i < d ? q_s[i] : 0.f;
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[r][e] = fmaf(k, u[e], s[r][e]);
                    acc[e] = fmaf(s[r][e], q, acc[e]);
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) part_s[l.rg * dv + l.c0 + e] = acc[e];
        }
        __syncthreads();
        float o = 0.f;
        if (tid < dv)
            for (int r = 0; r < l.groups; ++r) o += part_s[r * dv + tid];
        o *= qf;
        const float tot = rst_block_sum(o * o, red);
        if (tid < dv) {
            const float z = g_s[tid];
            out[((size_t)t * H + h) * dv + tid] = from_f32<T>(o * (1.0f / sqrtf(tot / (float)dv + eps)) * norm_w[tid] * (z / (1.0f + expf(-z))));
        }
        __syncthreads();                              // the next token overwrites the shared rows
    }
    if (mine) {
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            const int i = l.rg + r * l.groups;
            if (i < d) rst_store<VEC>(Sg + (size_t)i * dv + l.c0, s[r]);
        }
    }
}

// whether the kernel holds a head's state: rows of a thread
static int dh_rows(int d, int dv, int vec) { return (d + RST_THREADS / (dv / vec) - 1) / (RST_THREADS / (dv / vec)); }

KESTREL_API int kestrel_delta_head_step_takes(int d, int dv) { return d > 0 && dv > 0 && d <= 256 && dv <= 256 && dv % 4 == 0 && dh_rows(d, dv, 4) <= 32; }

KESTREL_API int kestrel_delta_head_step(const float *partial, int S, long long slice_stride, int ld, int col_g, int col_beta, int col_a, const float *conv_w,
                                        int taps, const float *A_log, const float *dt_bias, const float *norm_w, float eps, float *state,
                                        long long state_stride, long long tail_off, const int *cu_seqlens, const int *slots, void *out, int dtype, int nseq,
                                        int H, int G, int d, int dv, cudaStream_t stream) {
    if (nseq == 0) return 0;
    KESTREL_REQUIRE(nseq > 0 && nseq <= 65535 && S > 0 && H > 0 && G > 0 && H % G == 0 && kestrel_delta_head_step_takes(d, dv) && taps >= 1 && taps <= 9 &&
                    tail_off >= (long long)H * d * dv && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0, "delta_head_step: bad sizes H=%d d=%d dv=%d", H, d, dv);
    const int rows = dh_rows(d, dv, 4);
#define DH_GO(TT, R) kestrel_launch(delta_head_step_kernel<TT, 4, R>, dim3(H, nseq), dim3(RST_THREADS), 0, stream, partial, S, (size_t)slice_stride, ld, col_g, \
                                    col_beta, col_a, conv_w, taps, A_log, dt_bias, norm_w, eps, state, (size_t)state_stride, (size_t)tail_off, cu_seqlens, slots, \
                                    (TT *)out, H, G, d, dv)
#define DH_ROWS(TT) { if (rows <= 4) DH_GO(TT, 4); else if (rows <= 8) DH_GO(TT, 8); else if (rows <= 16) DH_GO(TT, 16); else DH_GO(TT, 32); }
    if (dtype == KESTREL_F32) DH_ROWS(float)
    else if (dtype == KESTREL_BF16) DH_ROWS(__nv_bfloat16)
    else return kestrel_fail(-2, "delta_head_step: unknown dtype %d", dtype);
#undef DH_ROWS
#undef DH_GO
    int rc = kestrel_check_launch("delta_head_step");
    if (rc) return rc;
    return kestrel_short_conv_tail(partial, S, slice_stride, ld, 0, taps, state, state_stride, tail_off, cu_seqlens, slots, nseq, 2 * G * d + H * dv, stream);
}
