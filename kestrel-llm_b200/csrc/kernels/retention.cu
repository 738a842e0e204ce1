// Retention: linear attention with a fixed decay per head.  Per head, with d key and dv value channels,
//
//   S_t = decay S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t
//
// q and k rotated by position (rotate-half pairs of a head's first `rot` dimensions), k times d^-1/2 afterwards.  S is float32,
// [d, dv] a head, in the request's state slot.
//
// Three ways through it, by the most tokens a request brings in a step:
//   few     retention_step: a CTA a (request, head) does everything between the fused product and the output product - q, k, v out
//           of the product's slices, the rotation, the state's update and read-out in one pass over it, the head's norm, the gate;
//   many    (bfloat16) chunks of 64 tokens on the tensor cores.  With g the decay and a chunk's tokens numbered 0 .. n - 1,
//             o_i = g^(i+1) S^T q_i + sum_{j <= i} g^(i-j) (q_i . k_j) v_j,      S' = g^n S + sum_j g^(n-1-j) k_j v_j^T
//           chunk_kv makes every chunk's sum over k_j v_j^T, chunk_scan runs the chunks of a request in order and leaves the state
//           in front of each, chunk_out makes the outputs, norms and gates them.  q, k, v are the bfloat16 operands the projections
//           give; what the recurrence itself makes - the decays' powers, decayed values, the state, the masked scores - is float32,
//           and enters a product as TWO bfloat16 terms (the rounded value and the rest), 16 bits of mantissa together;
//   between (and float32) retention_prepare and the sequential scan of linear_recurrence.cu.
#include "common.cuh"
#include "mma_sync.cuh"
#include <math.h>

#define RT_WARPS 4

// ---- what enters the recurrence, from the columns [q: H d | k: H d | v: H dv | ...] of a fused product ---------------------------
// A warp a head row; q, k, v in the type of the outputs; `w_out`, where given, receives the head's decay in every key channel.
template <typename T>
__global__ void __launch_bounds__(RT_WARPS * 32)
retention_prepare_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, const int *__restrict__ positions,
                         const float *__restrict__ inv_freq, int rot, const float *__restrict__ decay, T *__restrict__ q_out,
                         T *__restrict__ k_out, T *__restrict__ v_out, float *__restrict__ w_out, int H, int d, int dv) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float pos = (float)positions[t], k_scale = 1.0f / sqrtf((float)d);
    const int half = rot / 2;
    for (int r = blockIdx.y * RT_WARPS + warp; r < 3 * H; r += gridDim.y * RT_WARPS) {
        const int kind = r / H, h = r % H;                    // 0 q, 1 k, 2 v
        if (kind == 2) {
            const size_t col0 = (size_t)t * ld + 2 * (size_t)H * d + (size_t)h * dv;
            for (int i = lane; i < dv; i += 32) v_out[((size_t)t * H + h) * dv + i] = from_f32<T>(sum_slices(p, S, slice_stride, col0 + i));
            continue;
        }
        const size_t col0 = (size_t)t * ld + (size_t)kind * H * d + (size_t)h * d, o0 = ((size_t)t * H + h) * d;
        T *dst = kind == 0 ? q_out : k_out;
        const float mul = kind == 0 ? 1.0f : k_scale;
        for (int i = lane; i < half; i += 32) {               // both members of a pair
            const float u = sum_slices(p, S, slice_stride, col0 + i), v = sum_slices(p, S, slice_stride, col0 + half + i);
            float sn, cs;
            sincosf(pos * inv_freq[i], &sn, &cs);
            dst[o0 + i] = from_f32<T>((u * cs - v * sn) * mul);
            dst[o0 + half + i] = from_f32<T>((v * cs + u * sn) * mul);
        }
        for (int i = rot + lane; i < d; i += 32) dst[o0 + i] = from_f32<T>(sum_slices(p, S, slice_stride, col0 + i) * mul);
        if (w_out && kind == 0) {
            const float g = decay[h];
            for (int i = lane; i < d; i += 32) w_out[o0 + i] = g;
        }
    }
}

// The same where all of a head is turned and the sizes are multiples of 8: a thread takes eight numbers, four of a head's first half
// with their partners, or eight of the values.  Same bits.
__device__ __forceinline__ void rp_store4(float *dst, const float (&x)[4]) { *reinterpret_cast<float4 *>(dst) = make_float4(x[0], x[1], x[2], x[3]); }
__device__ __forceinline__ void rp_store4(__nv_bfloat16 *dst, const float (&x)[4]) { *reinterpret_cast<uint2 *>(dst) = make_uint2(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3])); }

template <typename T>
__global__ void __launch_bounds__(256)
retention_prepare_rows_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, const int *__restrict__ positions,
                              const float *__restrict__ inv_freq, const float *__restrict__ decay, T *__restrict__ q_out, T *__restrict__ k_out,
                              T *__restrict__ v_out, float *__restrict__ w_out, int H, int d, int dv) {
    __shared__ float cs_s[128], sn_s[128];
    pdl_launch_dependents();
    const int t = blockIdx.x, tid = threadIdx.x, half = d / 2, per = d / 8, n_qk = H * per, n = 2 * n_qk + H * dv / 8;
    const float pos = (float)positions[t], k_scale = 1.0f / sqrtf((float)d);
    for (int i = tid; i < half; i += 256) sincosf(pos * inv_freq[i], &sn_s[i], &cs_s[i]);
    __syncthreads();
    pdl_wait();
    for (int u = tid; u < n; u += 256) {
        const bool is_v = u >= 2 * n_qk, is_k = !is_v && u >= n_qk;
        const int w = is_k ? u - n_qk : u, h = is_v ? 0 : w / per, j = is_v ? 0 : w % per;
        const size_t col = is_v ? 2 * (size_t)H * d + (size_t)(u - 2 * n_qk) * 8 : (is_k ? (size_t)H * d : 0) + (size_t)h * d + 4 * j;
        const int other = is_v ? 4 : half;
        float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
        const float *src = p + (size_t)t * ld + col;
#pragma unroll 4
        for (int s = 0; s < S; ++s) {
            const float4 x = *reinterpret_cast<const float4 *>(src + (size_t)s * slice_stride), y = *reinterpret_cast<const float4 *>(src + (size_t)s * slice_stride + other);
            a[0] += x.x; a[1] += x.y; a[2] += x.z; a[3] += x.w;
            b[0] += y.x; b[1] += y.y; b[2] += y.z; b[3] += y.w;
        }
        if (is_v) {
            T *dst = v_out + (size_t)t * H * dv + (size_t)(u - 2 * n_qk) * 8;
            rp_store4(dst, a);
            rp_store4(dst + 4, b);
            continue;
        }
        const float mul = is_k ? k_scale : 1.0f;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const float x = a[c], y = b[c], cs = cs_s[4 * j + c], sn = sn_s[4 * j + c];
            a[c] = (x * cs - y * sn) * mul;
            b[c] = (y * cs + x * sn) * mul;
        }
        T *dst = (is_k ? k_out : q_out) + ((size_t)t * H + h) * d + 4 * j;
        rp_store4(dst, a);
        rp_store4(dst + half, b);
        if (w_out && !is_k) {
            const float g = decay[h];
            float *wd = w_out + ((size_t)t * H + h) * d + 4 * j;
            const float gg[4] = {g, g, g, g};
            rp_store4(wd, gg);
            rp_store4(wd + half, gg);
        }
    }
}

KESTREL_API int kestrel_retention_prepare(const float *partial, int S, long long slice_stride, int ld, const int *positions, const float *inv_freq,
                                          int rot, const float *decay, void *q_out, void *k_out, void *v_out, float *w_out, int dtype, int T, int H,
                                          int d, int dv, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && S > 0 && H > 0 && d > 0 && dv > 0 && ld >= H * (2 * d + dv), "retention_prepare: bad sizes");
    KESTREL_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= d && (rot == 0 || inv_freq), "retention_prepare: %d rotated dimensions of a head of %d", rot, d);
    if (rot == d && d % 8 == 0 && d <= 256 && dv % 8 == 0 && ld % 4 == 0 && slice_stride % 4 == 0 && ((uintptr_t)partial & 15) == 0) {
        if (dtype == KESTREL_F32)
            kestrel_launch(retention_prepare_rows_kernel<float>, dim3(T), dim3(256), 0, stream, partial, S, (size_t)slice_stride, ld, positions, inv_freq, decay,
                           (float *)q_out, (float *)k_out, (float *)v_out, w_out, H, d, dv);
        else if (dtype == KESTREL_BF16)
            kestrel_launch(retention_prepare_rows_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, partial, S, (size_t)slice_stride, ld, positions, inv_freq,
                           decay, (__nv_bfloat16 *)q_out, (__nv_bfloat16 *)k_out, (__nv_bfloat16 *)v_out, w_out, H, d, dv);
        else
            return kestrel_fail(-2, "retention_prepare: unknown dtype %d", dtype);
        return kestrel_check_launch("retention_prepare");
    }
    const int by = T >= 512 ? 1 : (3 * H + RT_WARPS - 1) / RT_WARPS;
    if (dtype == KESTREL_F32)
        kestrel_launch(retention_prepare_kernel<float>, dim3(T, by), dim3(RT_WARPS * 32), 0, stream, partial, S, (size_t)slice_stride, ld, positions, inv_freq,
                       rot, decay, (float *)q_out, (float *)k_out, (float *)v_out, w_out, H, d, dv);
    else if (dtype == KESTREL_BF16)
        kestrel_launch(retention_prepare_kernel<__nv_bfloat16>, dim3(T, by), dim3(RT_WARPS * 32), 0, stream, partial, S, (size_t)slice_stride, ld, positions,
                       inv_freq, rot, decay, (__nv_bfloat16 *)q_out, (__nv_bfloat16 *)k_out, (__nv_bfloat16 *)v_out, w_out, H, d, dv);
    else
        return kestrel_fail(-2, "retention_prepare: unknown dtype %d", dtype);
    return kestrel_check_launch("retention_prepare");
}

// ---- a step of few tokens ------------------------------------------------------------------------------------------------------
#define RS_THREADS 256
template <typename T, int VEC>
__global__ void __launch_bounds__(RS_THREADS)
retention_step_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, const int *__restrict__ positions,
                      const float *__restrict__ inv_freq, int rot, const float *__restrict__ decay, float *__restrict__ state, size_t state_stride,
                      size_t state_off, const int *__restrict__ cu_seqlens, const int *__restrict__ slots, float eps, T *__restrict__ out, int H,
                      int d, int dv) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float q_s[256], k_s[256], v_s[256], g_s[256];
    __shared__ float part_s[RS_THREADS * VEC];        // [row group][dv]
    __shared__ float red[RS_THREADS / 32];
    const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1];
    if (t0 == t1) return;
    float *Sg = state + (size_t)slots[seq] * state_stride + state_off + (size_t)h * d * dv;
    const float g = decay[h], k_scale = 1.0f / sqrtf((float)d);
    const int half = rot / 2, n_pass = d - rot;
    const int cols = dv / VEC, groups = RS_THREADS / cols;          // a thread: VEC columns, every groups-th key channel
    const int rg = tid / cols, c0 = tid % cols * VEC;
    for (int t = t0; t < t1; ++t) {
        const size_t row = (size_t)t * ld;
        const float pos = (float)positions[t];
        // the threads of a token: pairs of q, pairs of k, channels of q and k that pass, values, gate logits
        const int n_all = 2 * half + 2 * n_pass + 2 * dv;
        for (int u = tid; u < n_all; u += RS_THREADS) {
            if (u < 2 * half) {
                const bool is_k = u >= half;
                const int i = is_k ? u - half : u;
                const size_t col = row + (is_k ? (size_t)H * d : 0) + (size_t)h * d + i;
                const float a = sum_slices(p, S, slice_stride, col), b = sum_slices(p, S, slice_stride, col + half);
                float sn, cs;
                sincosf(pos * inv_freq[i], &sn, &cs);
                const float mul = is_k ? k_scale : 1.0f;
                float *dst = is_k ? k_s : q_s;
                dst[i] = (a * cs - b * sn) * mul;
                dst[half + i] = (b * cs + a * sn) * mul;
            } else if (u < 2 * half + 2 * n_pass) {
                const int w = u - 2 * half;
                const bool is_k = w >= n_pass;
                const int i = rot + (is_k ? w - n_pass : w);
                const float a = sum_slices(p, S, slice_stride, row + (is_k ? (size_t)H * d : 0) + (size_t)h * d + i);
                if (is_k) k_s[i] = a * k_scale;
                else q_s[i] = a;
            } else {
                const int w = u - 2 * half - 2 * n_pass;
                const bool is_g = w >= dv;
                const int i = is_g ? w - dv : w;
                const float a = sum_slices(p, S, slice_stride, row + 2 * (size_t)H * d + (is_g ? (size_t)H * dv : 0) + (size_t)h * dv + i);
                if (is_g) g_s[i] = a;
                else v_s[i] = a;
            }
        }
        __syncthreads();
        float acc[VEC], v[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            acc[e] = 0.f;
            v[e] = rg < groups ? v_s[c0 + e] : 0.f;
        }
        if (rg < groups) {
            for (int i0 = rg; i0 < d; i0 += 8 * groups) {            // eight rows' loads in flight
                __align__(16) float s[8][VEC];
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    const int i = i0 + r * groups;
                    if (i >= d) continue;
                    if (VEC == 4) *reinterpret_cast<float4 *>(s[r]) = *reinterpret_cast<const float4 *>(Sg + (size_t)i * dv + c0);
                    else s[r][0] = Sg[(size_t)i * dv + c0];
                }
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    const int i = i0 + r * groups;
                    if (i >= d) continue;
                    const float ki = k_s[i], qi = q_s[i];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        s[r][e] = fmaf(g, s[r][e], ki * v[e]);
                        acc[e] = fmaf(s[r][e], qi, acc[e]);
                    }
                    if (VEC == 4) *reinterpret_cast<float4 *>(Sg + (size_t)i * dv + c0) = *reinterpret_cast<const float4 *>(s[r]);
                    else Sg[(size_t)i * dv + c0] = s[r][0];
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) part_s[rg * dv + c0 + e] = acc[e];
        }
        __syncthreads();
        float o = 0.f;                                // dv <= RS_THREADS: a thread a value channel
        if (tid < dv)
            for (int r = 0; r < groups; ++r) o += part_s[r * dv + tid];
        const float ss = warp_sum(o * o);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        float tot = 0.f;
#pragma unroll
        for (int w = 0; w < RS_THREADS / 32; ++w) tot += red[w];
        if (tid < dv) {
            const float z = g_s[tid];
            out[((size_t)t * H + h) * dv + tid] = from_f32<T>(o * (1.0f / sqrtf(tot / (float)dv + eps)) * (z / (1.0f + expf(-z))));
        }
        __syncthreads();                              // the next token overwrites the shared rows; this thread's state rows are its own
    }
}

KESTREL_API int kestrel_retention_step(const float *partial, int S, long long slice_stride, int ld, const int *positions, const float *inv_freq,
                                       int rot, const float *decay, float *state, long long state_stride, long long state_off,
                                       const int *cu_seqlens, const int *slots, float eps, void *out, int dtype, int nseq, int H, int d, int dv,
                                       cudaStream_t stream) {
    if (nseq == 0) return 0;
    KESTREL_REQUIRE(nseq > 0 && nseq <= 65535 && S > 0 && H > 0 && d > 0 && d <= 256 && dv > 0 && dv <= 256 && state_off >= 0 && ld >= 2 * H * (d + dv),
                    "retention_step: bad sizes H=%d d=%d dv=%d", H, d, dv);
    KESTREL_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= d && (rot == 0 || inv_freq), "retention_step: %d rotated dimensions of a head of %d", rot, d);
    const bool vec = dv % 4 == 0 && state_stride % 4 == 0 && state_off % 4 == 0 && ((uintptr_t)state & 15) == 0;
#define RS_LAUNCH(TT, V) kestrel_launch(retention_step_kernel<TT, V>, dim3(H, nseq), dim3(RS_THREADS), 0, stream, partial, S, (size_t)slice_stride, ld, positions, \
                                        inv_freq, rot, decay, state, (size_t)state_stride, (size_t)state_off, cu_seqlens, slots, eps, (TT *)out, H, d, dv)
    if (dtype == KESTREL_F32) { if (vec) RS_LAUNCH(float, 4); else RS_LAUNCH(float, 1); }
    else if (dtype == KESTREL_BF16) { if (vec) RS_LAUNCH(__nv_bfloat16, 4); else RS_LAUNCH(__nv_bfloat16, 1); }
    else return kestrel_fail(-2, "retention_step: unknown dtype %d", dtype);
#undef RS_LAUNCH
    return kestrel_check_launch("retention_step");
}

// ---- chunks of many tokens ---------------------------------------------------------------------------------------------------
#define RC_C 64                  // tokens of a chunk
#define RC_N 64                  // value columns worked on at a time
#define RC_LDN (RC_N + 8)        // row lengths in shared memory that keep ldmatrix free of bank conflicts

struct RetentionChunkParams {
    const __nv_bfloat16 *q, *k, *v;      // [T, H d], [T, H d], [T, H dv]
    const float *powers;                 // [H, RC_C + 1]
    const int *cu_seqlens, *slots, *tile_seq, *tile_row0, *first_tile;
    float *state, *scratch;              // scratch [tiles, H, d, dv]: the chunks' sums
    __nv_bfloat16 *before;               // [tiles, H, 2, d, dv]: the states in front of the chunks, as two terms
    size_t state_stride, state_off;
    const float *gate;                   // the fused product
    int gate_slices, gate_ld, gate_col0;
    size_t gate_stride;
    float eps;
    __nv_bfloat16 *out;
    int H, d, dv;
};

// two bfloat16 terms of a float32: the rounded value and what it leaves
__device__ __forceinline__ void rc_split(float x, __nv_bfloat16 &hi, __nv_bfloat16 &lo) {
    hi = __float2bfloat16_rn(x);
    lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}
__device__ __forceinline__ uint32_t rc_bits(__nv_bfloat16 a, __nv_bfloat16 b) {
    __nv_bfloat162 v;
    v.x = a;
    v.y = b;
    return *reinterpret_cast<uint32_t *>(&v);
}

__device__ __forceinline__ void rc_cp16(__nv_bfloat16 *dst, const __nv_bfloat16 *src, bool valid) {
    const int sz = valid ? 16 : 0;                    // 0: sixteen zero bytes
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(sz) : "memory");
}

// a chunk's rows of a head into shared memory [RC_C][D + 8], zero beyond its tokens and channels
template <int D>
__device__ __forceinline__ void rc_load_rows(__nv_bfloat16 *dst, const __nv_bfloat16 *src, size_t row_stride, int n, int d, int tid) {
    for (int idx = tid; idx < RC_C * (D / 8); idx += 128) {
        const int r = idx / (D / 8), c = idx % (D / 8) * 8;
        const bool ok = r < n && c < d;
        rc_cp16(dst + r * (D + 8) + c, src + (ok ? (size_t)r * row_stride + c : 0), ok);
    }
}

// scratch[tile, h] = sum_j g^(n-1-j) k_j v_j^T, columns [64 z, 64 z + 64)
template <int D>
__global__ void __launch_bounds__(128)
retention_chunk_kv_kernel(const RetentionChunkParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t rc_smem[];
    __nv_bfloat16 *Ks = reinterpret_cast<__nv_bfloat16 *>(rc_smem), *Vh = Ks + RC_C * (D + 8), *Vl = Vh + RC_C * RC_LDN;
    const int tile = blockIdx.x, h = blockIdx.y, n0 = blockIdx.z * RC_N, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = p.tile_seq[tile], row0 = p.tile_row0[tile], tb = p.cu_seqlens[seq], n = min(RC_C, p.cu_seqlens[seq + 1] - tb - row0);
    const int d = p.d, dv = p.dv;
    const size_t t0 = (size_t)tb + row0;
    const float *pw = p.powers + (size_t)h * (RC_C + 1);
    rc_load_rows<D>(Ks, p.k + (t0 * p.H + h) * d, (size_t)p.H * d, n, d, tid);
    for (int idx = tid; idx < RC_C * (RC_N / 2); idx += 128) {
        const int r = idx / (RC_N / 2), c = idx % (RC_N / 2) * 2;
        __nv_bfloat16 h0 = __float2bfloat16_rn(0.f), h1 = h0, l0 = h0, l1 = h0;
        if (r < n && n0 + c < dv) {
            const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162 *>(p.v + ((t0 + r) * p.H + h) * dv + n0 + c);
            const float w = pw[n - 1 - r];
            rc_split(__bfloat162float(x.x) * w, h0, l0);
            rc_split(__bfloat162float(x.y) * w, h1, l1);
        }
        *reinterpret_cast<uint32_t *>(Vh + r * RC_LDN + c) = rc_bits(h0, h1);
        *reinterpret_cast<uint32_t *>(Vl + r * RC_LDN + c) = rc_bits(l0, l1);
    }
    asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int g = lane >> 2, tq = lane & 3;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_col = (lane >> 4) * 8;
    const int a_k = (lane & 7) + (lane >> 4) * 8, a_m = ((lane >> 3) & 1) * 8;           // K^T fragments: rows of memory are tokens
    float *dst = p.scratch + ((size_t)tile * p.H + h) * d * dv;
    for (int mt = warp; mt * 16 < d; mt += 4) {
        float acc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[j][c] = 0.f;
#pragma unroll
        for (int kk = 0; kk < RC_C / 16; ++kk) {
            uint32_t a[4];
            ldmatrix_x4_trans((uint32_t)__cvta_generic_to_shared(Ks + (kk * 16 + a_k) * (D + 8) + mt * 16 + a_m), a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int np = 0; np < RC_N / 16; ++np) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans((uint32_t)__cvta_generic_to_shared(Vh + (kk * 16 + v_row) * RC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(acc[2 * np], a, b0, b1);
                mma_bf16(acc[2 * np + 1], a, b2, b3);
                ldmatrix_x4_trans((uint32_t)__cvta_generic_to_shared(Vl + (kk * 16 + v_row) * RC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(acc[2 * np], a, b0, b1);
                mma_bf16(acc[2 * np + 1], a, b2, b3);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int col = n0 + j * 8 + 2 * tq;
            if (col >= dv) continue;
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int i = mt * 16 + g + 8 * hf;
                if (i < d) *reinterpret_cast<float2 *>(dst + (size_t)i * dv + col) = make_float2(acc[j][2 * hf], acc[j][2 * hf + 1]);
            }
        }
    }
}

// Per request and head: the state in front of every chunk, as the two terms its product takes, then the state after the last one.
__global__ void __launch_bounds__(256)
retention_chunk_scan_kernel(const RetentionChunkParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, seq = blockIdx.z, n4 = p.d * p.dv / 4, i = blockIdx.x * 256 + threadIdx.x;
    if (i >= n4) return;
    const int lo = p.first_tile[seq], hi = p.first_tile[seq + 1], tokens = p.cu_seqlens[seq + 1] - p.cu_seqlens[seq];
    if (lo == hi) return;
    const float *pw = p.powers + (size_t)h * (RC_C + 1);
    float4 *st = reinterpret_cast<float4 *>(p.state + (size_t)p.slots[seq] * p.state_stride + p.state_off + (size_t)h * p.d * p.dv) + i;
    const float4 *sc = reinterpret_cast<const float4 *>(p.scratch) + ((size_t)lo * p.H + h) * n4 + i;
    uint2 *bf = reinterpret_cast<uint2 *>(p.before) + ((size_t)lo * p.H + h) * 2 * n4 + i;
    const size_t step = (size_t)p.H * n4;
    float4 s = *st;
    const float full = pw[RC_C];
    for (int c = lo; c < hi; c += 8) {
        float4 kv[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (c + u < hi) kv[u] = sc[(size_t)(c - lo + u) * step];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            if (c + u >= hi) break;
            const float g = c + u + 1 < hi ? full : pw[tokens - (hi - 1 - lo) * RC_C];
            __nv_bfloat16 hi4[4], lo4[4];
            rc_split(s.x, hi4[0], lo4[0]);
            rc_split(s.y, hi4[1], lo4[1]);
            rc_split(s.z, hi4[2], lo4[2]);
            rc_split(s.w, hi4[3], lo4[3]);
            bf[(size_t)(c - lo + u) * 2 * step] = make_uint2(rc_bits(hi4[0], hi4[1]), rc_bits(hi4[2], hi4[3]));
            bf[(size_t)(c - lo + u) * 2 * step + n4] = make_uint2(rc_bits(lo4[0], lo4[1]), rc_bits(lo4[2], lo4[3]));
            s.x = fmaf(g, s.x, kv[u].x);
            s.y = fmaf(g, s.y, kv[u].y);
            s.z = fmaf(g, s.z, kv[u].z);
            s.w = fmaf(g, s.w, kv[u].w);
        }
    }
    *st = s;
}

// A chunk's outputs of a head: warp w has tokens 16 w .. 16 w + 15; NS slices of 64 value columns.
template <int D, int NS>
__global__ void __launch_bounds__(128)
retention_chunk_out_kernel(const RetentionChunkParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t rc_smem[];
    __nv_bfloat16 *Qs = reinterpret_cast<__nv_bfloat16 *>(rc_smem), *Ks = Qs + RC_C * (D + 8), *Vs = Ks + RC_C * (D + 8);
    __nv_bfloat16 *Sh = Vs + RC_C * RC_LDN, *Sl = Sh + D * RC_LDN;
    __shared__ float pw[RC_C + 1];
    const int tile = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = p.tile_seq[tile], row0 = p.tile_row0[tile], tb = p.cu_seqlens[seq], n = min(RC_C, p.cu_seqlens[seq + 1] - tb - row0);
    const int d = p.d, dv = p.dv, k_steps = (d + 15) / 16;
    const size_t t0 = (size_t)tb + row0;
    const __nv_bfloat16 *st = p.before + ((size_t)tile * p.H + h) * 2 * d * dv;
    auto load_slice = [&](int n0) {
        for (int idx = tid; idx < RC_C * (RC_N / 8); idx += 128) {
            const int r = idx / (RC_N / 8), c = idx % (RC_N / 8) * 8;
            const bool ok = r < n && n0 + c < dv;
            rc_cp16(Vs + r * RC_LDN + c, p.v + (ok ? ((t0 + r) * p.H + h) * dv + n0 + c : 0), ok);
        }
        for (int idx = tid; idx < D * (RC_N / 8); idx += 128) {
            const int i = idx / (RC_N / 8), c = idx % (RC_N / 8) * 8;
            const bool ok = i < d && n0 + c < dv;
            const size_t off = ok ? (size_t)i * dv + n0 + c : 0;
            rc_cp16(Sh + i * RC_LDN + c, st + off, ok);
            rc_cp16(Sl + i * RC_LDN + c, st + (size_t)d * dv + off, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    rc_load_rows<D>(Qs, p.q + (t0 * p.H + h) * d, (size_t)p.H * d, n, d, tid);
    rc_load_rows<D>(Ks, p.k + (t0 * p.H + h) * d, (size_t)p.H * d, n, d, tid);
    asm volatile("cp.async.commit_group;" ::: "memory");
    load_slice(0);                                    // under the scores
    for (int i = tid; i <= RC_C; i += 128) pw[i] = p.powers[(size_t)h * (RC_C + 1) + i];
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const int g = lane >> 2, tq = lane & 3;
    const int a_row = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, a_k = (lane >> 4) * 8;
    const int b_row = (lane & 7) + (lane >> 4) * 8, b_k = ((lane >> 3) & 1) * 8;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_col = (lane >> 4) * 8;
    // the scores of this warp's tokens with the chunk's, decayed and masked, as two terms in the layout of an A operand
    uint32_t ph[RC_C / 16][4], pl[RC_C / 16][4];
    {
        float s[RC_C / 8][4];
#pragma unroll
        for (int j = 0; j < RC_C / 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[j][c] = 0.f;
        for (int kk = 0; kk < k_steps; ++kk) {
            uint32_t a[4];
            ldmatrix_x4((uint32_t)__cvta_generic_to_shared(Qs + a_row * (D + 8) + kk * 16 + a_k), a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int jp = 0; jp < RC_C / 16; ++jp) {
                if (jp > warp) continue;              // keys behind the warp's last token
                uint32_t b00, b01, b10, b11;
                ldmatrix_x4((uint32_t)__cvta_generic_to_shared(Ks + (jp * 16 + b_row) * (D + 8) + kk * 16 + b_k), b00, b01, b10, b11);
                mma_bf16(s[2 * jp], a, b00, b01);
                mma_bf16(s[2 * jp + 1], a, b10, b11);
            }
        }
#pragma unroll
        for (int jp = 0; jp < RC_C / 16; ++jp)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                // register e of the operand: row g (+ 8), keys 2 tq (+ 8)
                const int jt = 2 * jp + (e >> 1), i = warp * 16 + g + 8 * (e & 1), j = jt * 8 + 2 * tq;
                const float x0 = i >= j ? s[jt][2 * (e & 1)] * pw[i - j] : 0.f, x1 = i > j ? s[jt][2 * (e & 1) + 1] * pw[i - j - 1] : 0.f;
                __nv_bfloat16 h0, h1, l0, l1;
                rc_split(x0, h0, l0);
                rc_split(x1, h1, l1);
                ph[jp][e] = rc_bits(h0, h1);
                pl[jp][e] = rc_bits(l0, l1);
            }
    }
    float o[NS][RC_N / 8][4];
#pragma unroll
    for (int ns = 0; ns < NS; ++ns) {
        if (ns > 0) {
            __syncthreads();                          // everyone has left the slice before
            load_slice(ns * RC_N);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        float (&oo)[RC_N / 8][4] = o[ns];
#pragma unroll
        for (int j = 0; j < RC_N / 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) oo[j][c] = 0.f;
        for (int kk = 0; kk < k_steps; ++kk) {
            uint32_t a[4];
            ldmatrix_x4((uint32_t)__cvta_generic_to_shared(Qs + a_row * (D + 8) + kk * 16 + a_k), a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int np = 0; np < RC_N / 16; ++np) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans((uint32_t)__cvta_generic_to_shared(Sh + (kk * 16 + v_row) * RC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(oo[2 * np], a, b0, b1);
                mma_bf16(oo[2 * np + 1], a, b2, b3);
                ldmatrix_x4_trans((uint32_t)__cvta_generic_to_shared(Sl + (kk * 16 + v_row) * RC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(oo[2 * np], a, b0, b1);
                mma_bf16(oo[2 * np + 1], a, b2, b3);
            }
        }
        const float g0 = pw[warp * 16 + g + 1], g1 = pw[warp * 16 + g + 9];
#pragma unroll
        for (int j = 0; j < RC_N / 8; ++j) {
            oo[j][0] *= g0;
            oo[j][1] *= g0;
            oo[j][2] *= g1;
            oo[j][3] *= g1;
        }
#pragma unroll
        for (int jp = 0; jp < RC_C / 16; ++jp) {
            if (jp > warp) continue;
#pragma unroll
            for (int np = 0; np < RC_N / 16; ++np) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans((uint32_t)__cvta_generic_to_shared(Vs + (jp * 16 + v_row) * RC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(oo[2 * np], ph[jp], b0, b1);
                mma_bf16(oo[2 * np + 1], ph[jp], b2, b3);
                mma_bf16(oo[2 * np], pl[jp], b0, b1);
                mma_bf16(oo[2 * np + 1], pl[jp], b2, b3);
            }
        }
    }
    // the head's norm (columns beyond dv are zero) and the gate
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        float ss = 0.f;
#pragma unroll
        for (int ns = 0; ns < NS; ++ns)
#pragma unroll
            for (int j = 0; j < RC_N / 8; ++j) {
                ss = fmaf(o[ns][j][2 * hf], o[ns][j][2 * hf], ss);
                ss = fmaf(o[ns][j][2 * hf + 1], o[ns][j][2 * hf + 1], ss);
            }
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        const int i = warp * 16 + g + 8 * hf;
        if (i >= n) continue;
        const float rn = 1.0f / sqrtf(ss / (float)dv + p.eps);
        const size_t gate_row = (t0 + i) * p.gate_ld + p.gate_col0 + (size_t)h * dv;
        __nv_bfloat16 *dst = p.out + ((t0 + i) * p.H + h) * dv;
        float2 z[NS][RC_N / 8];                       // all of a row's gate logits in flight at once
#pragma unroll
        for (int ns = 0; ns < NS; ++ns)
#pragma unroll
            for (int j = 0; j < RC_N / 8; ++j) z[ns][j] = make_float2(0.f, 0.f);
        for (int s = 0; s < p.gate_slices; ++s)
#pragma unroll
            for (int ns = 0; ns < NS; ++ns)
#pragma unroll
                for (int j = 0; j < RC_N / 8; ++j) {
                    const int col = ns * RC_N + j * 8 + 2 * tq;
                    if (col >= dv) continue;
                    const float2 x = *reinterpret_cast<const float2 *>(p.gate + (size_t)s * p.gate_stride + gate_row + col);
                    z[ns][j].x += x.x;
                    z[ns][j].y += x.y;
                }
#pragma unroll
        for (int ns = 0; ns < NS; ++ns)
#pragma unroll
            for (int j = 0; j < RC_N / 8; ++j) {
                const int col = ns * RC_N + j * 8 + 2 * tq;
                if (col >= dv) continue;
                const float z0 = z[ns][j].x, z1 = z[ns][j].y;
                *reinterpret_cast<uint32_t *>(dst + col) = pack_bf16(o[ns][j][2 * hf] * rn * (z0 / (1.0f + expf(-z0))), o[ns][j][2 * hf + 1] * rn * (z1 / (1.0f + expf(-z1))));
            }
    }
}

KESTREL_API int kestrel_retention_chunk_tokens(void) { return RC_C; }

template <int D, int NS>
static int rc_launch(const RetentionChunkParams &p, int tiles, int nseq, cudaStream_t stream) {
    const size_t kv_smem = (size_t)RC_C * (D + 8 + 2 * RC_LDN) * 2, out_smem = (size_t)(RC_C * (2 * (D + 8) + RC_LDN) + 2 * D * RC_LDN) * 2;
    static bool attr_set = false;
    if (!attr_set) {
        if (cudaFuncSetAttribute(retention_chunk_kv_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kv_smem) != cudaSuccess ||
            cudaFuncSetAttribute(retention_chunk_out_kernel<D, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_smem) != cudaSuccess)
            return kestrel_fail(-3, "retention_chunks: cannot set the shared memory size");
        attr_set = true;
    }
    kestrel_launch(retention_chunk_kv_kernel<D>, dim3(tiles, p.H, NS), dim3(128), kv_smem, stream, p);
    int rc = kestrel_check_launch("retention_chunk_kv");
    if (rc) return rc;
    kestrel_launch(retention_chunk_scan_kernel, dim3((p.d * p.dv / 4 + 255) / 256, p.H, nseq), dim3(256), 0, stream, p);
    if ((rc = kestrel_check_launch("retention_chunk_scan"))) return rc;
    kestrel_launch(retention_chunk_out_kernel<D, NS>, dim3(tiles, p.H), dim3(128), out_smem, stream, p);
    return kestrel_check_launch("retention_chunk_out");
}

KESTREL_API int kestrel_retention_chunks(const void *q, const void *k, const void *v, const float *powers, const float *partial, int S,
                                         long long slice_stride, int ld, int gate_col0, float *state, long long state_stride, long long state_off,
                                         const int *cu_seqlens, const int *slots, const int *tile_seq, const int *tile_row0, const int *first_tile,
                                         int tiles, float *scratch, float eps, void *out, int nseq, int H, int d, int dv, cudaStream_t stream) {
    if (nseq == 0 || tiles == 0) return 0;
    KESTREL_REQUIRE(nseq > 0 && nseq <= 65535 && tiles > 0 && H > 0 && H <= 65535 && d > 0 && dv > 0 && d % 8 == 0 && dv % 8 == 0 && d <= 256 && dv <= 256,
                    "retention_chunks: bad sizes H=%d d=%d dv=%d", H, d, dv);
    KESTREL_REQUIRE(S > 0 && gate_col0 >= 0 && gate_col0 + H * dv <= ld && state_stride % 4 == 0 && state_off % 4 == 0 && ((uintptr_t)state & 15) == 0 && ld % 2 == 0 && gate_col0 % 2 == 0 && slice_stride % 2 == 0,
                    "retention_chunks: the gate's columns or the state's place do not fit");
    RetentionChunkParams p = {};
    p.q = (const __nv_bfloat16 *)q; p.k = (const __nv_bfloat16 *)k; p.v = (const __nv_bfloat16 *)v;
    p.powers = powers; p.cu_seqlens = cu_seqlens; p.slots = slots; p.tile_seq = tile_seq; p.tile_row0 = tile_row0; p.first_tile = first_tile;
    p.state = state; p.scratch = scratch; p.before = (__nv_bfloat16 *)(scratch + (size_t)tiles * H * d * dv); p.state_stride = (size_t)state_stride; p.state_off = (size_t)state_off;
    p.gate = partial; p.gate_slices = S; p.gate_ld = ld; p.gate_col0 = gate_col0; p.gate_stride = (size_t)slice_stride;
    p.eps = eps; p.out = (__nv_bfloat16 *)out; p.H = H; p.d = d; p.dv = dv;
#define RC_CASE(D)                                                              \
    do {                                                                        \
        if (dv <= 64) return rc_launch<D, 1>(p, tiles, nseq, stream);           \
        if (dv <= 128) return rc_launch<D, 2>(p, tiles, nseq, stream);          \
        return rc_launch<D, 4>(p, tiles, nseq, stream);                         \
    } while (0)
    if (d <= 32) RC_CASE(32);
    if (d <= 64) RC_CASE(64);
    if (d <= 128) RC_CASE(128);
    RC_CASE(256);
#undef RC_CASE
}
