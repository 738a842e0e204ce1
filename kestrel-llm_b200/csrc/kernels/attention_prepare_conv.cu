// The step between a fused query/key product and attention, for mixers whose queries and keys pass a short causal convolution and
// whose values ARE their keys:
//
//   u[t, c] = sum_j w[j, c] x[t - (taps - 1) + j, c]        per column of [q: nq hd | k: nkv hd]; inputs before a request's first
//                                                           token of this step from its state slot (as in short_conv.cu)
//   v = u_k as it is, into the V pages;   q, k = u / sqrt(mean(u^2) + eps) * weight [hd] per head, then the first `rot`
//   dimensions turned by position in rotate-half pairs (times `rot_scale`); q to its rows, k into the K pages.
//
// A warp takes a head row and a run of tokens, the convolution's inputs in registers; the block makes its tokens' cosines once.
// Everything is float32; a token's result depends on its inputs alone, not on the cut or the batch.
#include "common.cuh"
#include <math.h>

#define APC_WARPS 8
#define APC_RUN 4

template <typename T, int PER, int TP>
__global__ void __launch_bounds__(APC_WARPS * 32)
attn_prepare_conv_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, const float *__restrict__ conv_w, int taps,
                         const float *__restrict__ q_w, const float *__restrict__ k_w, float eps, const float *__restrict__ inv_freq, int rot,
                         float rot_scale, const float *__restrict__ state, size_t state_stride, size_t tail_off, const int *__restrict__ positions,
                         const int *__restrict__ seq_of_token, const int *__restrict__ cu_seqlens, const int *__restrict__ slots,
                         const int *__restrict__ block_table, int table_stride, int page_size, T *__restrict__ k_cache, T *__restrict__ v_cache,
                         T *__restrict__ q_out, int n_tokens, int nq, int nkv, int hd, int run) {
    __shared__ float cs_s[APC_RUN][128], sn_s[APC_RUN][128];
    __shared__ float pair_s[APC_WARPS][32 * PER];
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = rot / 2;
    const int t0 = blockIdx.x * run, t1 = min(t0 + run, n_tokens);
    for (int i = threadIdx.x; i < (t1 - t0) * half; i += APC_WARPS * 32) {     // the step's description is not the predecessor's output
        float sn, cs;
        sincosf((float)positions[t0 + i / half] * inv_freq[i % half], &sn, &cs);
        cs_s[i / half][i % half] = cs * rot_scale;
        sn_s[i / half][i % half] = sn * rot_scale;
    }
    __syncthreads();
    pdl_wait();
    const int C = (nq + nkv) * hd;
    for (int r = blockIdx.y * APC_WARPS + warp; r < nq + nkv; r += gridDim.y * APC_WARPS) {
        const bool is_k = r >= nq;
        const int head = is_k ? r - nq : r;
        const float *nw = is_k ? k_w : q_w;
        float f[TP][PER], x[TP][PER], w[PER];
#pragma unroll
        for (int c = 0; c < PER; ++c) {
            const int i = lane + 32 * c;
            w[c] = i < hd && nw ? nw[i] : 1.f;
#pragma unroll
            for (int j = 0; j < TP; ++j) f[j][c] = i < hd && j >= TP - taps ? conv_w[(size_t)(j - (TP - taps)) * C + (size_t)r * hd + i] : 0.f;
        }
        auto load = [&](float (&v)[PER], int t) {
#pragma unroll
            for (int c = 0; c < PER; ++c) v[c] = 0.f;
            const float *row = p + (size_t)t * ld + (size_t)r * hd;
#pragma unroll 4
            for (int s = 0; s < S; ++s)
#pragma unroll
                for (int c = 0; c < PER; ++c) {
                    const int i = lane + 32 * c;
                    if (i < hd) v[c] += row[(size_t)s * slice_stride + i];
                }
        };
        int seq = -1;
        for (int t = t0; t < t1; ++t) {
            const int q = seq_of_token[t];
            if (q != seq) {
                seq = q;
                const int first = cu_seqlens[q];
                const float *tail = state + (size_t)slots[q] * state_stride + tail_off;
#pragma unroll
                for (int j = 0; j < TP - 1; ++j) {
                    const int n = t - first - (TP - 1) + j;
                    if (j >= TP - taps && n >= 0) {
                        load(x[j], first + n);
                    } else {
#pragma unroll
                        for (int c = 0; c < PER; ++c) {
                            const int i = lane + 32 * c;
                            x[j][c] = j >= TP - taps && i < hd ? tail[(size_t)(taps - 1 + n) * C + (size_t)r * hd + i] : 0.f;
                        }
                    }
                }
            }
            load(x[TP - 1], t);
            float y[PER], ss = 0.f;
#pragma unroll
            for (int c = 0; c < PER; ++c) {
                y[c] = 0.f;
#pragma unroll
                for (int j = 0; j < TP; ++j) y[c] = fmaf(f[j][c], x[j][c], y[c]);
                ss = fmaf(y[c], y[c], ss);
            }
            T *dst;
            if (is_k) {
                const int pos = positions[t], page = block_table[(size_t)q * table_stride + pos / page_size];
                const size_t slot = (((size_t)page * nkv + head) * page_size + pos % page_size) * hd;
                dst = k_cache + slot;
#pragma unroll
                for (int c = 0; c < PER; ++c) {
                    const int i = lane + 32 * c;
                    if (i < hd) v_cache[slot + i] = from_f32<T>(y[c]);
                }
            } else {
                dst = q_out + ((size_t)t * nq + head) * hd;
            }
            const float mul = 1.0f / sqrtf(warp_sum(ss) / (float)hd + eps);
#pragma unroll
            for (int c = 0; c < PER; ++c) y[c] *= mul * w[c];
            if (rot > 0) {
#pragma unroll
                for (int c = 0; c < PER; ++c) pair_s[warp][lane + 32 * c] = y[c];
                __syncwarp();
#pragma unroll
                for (int c = 0; c < PER; ++c) {
                    const int i = lane + 32 * c;
                    if (i < rot) {
                        const int j = i < half ? i : i - half;
                        const float other = pair_s[warp][i < half ? i + half : i - half], cs = cs_s[t - t0][j], sn = sn_s[t - t0][j];
                        y[c] = i < half ? y[c] * cs - other * sn : y[c] * cs + other * sn;
                    }
                }
                __syncwarp();
            }
#pragma unroll
            for (int c = 0; c < PER; ++c) {
                const int i = lane + 32 * c;
                if (i < hd) dst[i] = from_f32<T>(y[c]);
            }
#pragma unroll
            for (int j = 0; j + 1 < TP; ++j)
#pragma unroll
                for (int c = 0; c < PER; ++c) x[j][c] = x[j + 1][c];
        }
    }
}

// The same where a head's size is 32, 64 or 128 and all of it is turned, or none: HD / 8 lanes take a head row, a lane the numbers
// 4 j .. 4 j + 3 and their partners HD / 2 + 4 j .., so that loads and stores are vectors and a pair is turned inside a lane; all inputs of
// a run of tokens are in flight together.
#define APF_THREADS 128
template <int N> struct ApfCount { static constexpr int value = N; };
__device__ __forceinline__ void apf_store4(float *dst, const float *x) { *reinterpret_cast<float4 *>(dst) = make_float4(x[0], x[1], x[2], x[3]); }
__device__ __forceinline__ void apf_store4(__nv_bfloat16 *dst, const float *x) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(x[0], x[1]), hi = __floats2bfloat162_rn(x[2], x[3]);
    *reinterpret_cast<uint2 *>(dst) = make_uint2(*reinterpret_cast<uint32_t *>(&lo), *reinterpret_cast<uint32_t *>(&hi));
}

template <typename T, int HD, int TP, int RUN>
__global__ void __launch_bounds__(APF_THREADS)
attn_prepare_conv_rows_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, const float *__restrict__ conv_w, int taps,
                              const float *__restrict__ q_w, const float *__restrict__ k_w, float eps, const float *__restrict__ inv_freq, int rot,
                              float rot_scale, const float *__restrict__ state, size_t state_stride, size_t tail_off, const int *__restrict__ positions,
                              const int *__restrict__ seq_of_token, const int *__restrict__ cu_seqlens, const int *__restrict__ slots,
                              const int *__restrict__ block_table, int table_stride, int page_size, T *__restrict__ k_cache, T *__restrict__ v_cache,
                              T *__restrict__ q_out, int n_tokens, int nq, int nkv) {
    constexpr int LANES = HD / 8, ROWS = APF_THREADS / LANES, HALF = HD / 2;
    __shared__ float cs_s[RUN][HALF], sn_s[RUN][HALF];
    pdl_launch_dependents();
    // the step's description and the weights are not the predecessor's output
    const int tid = threadIdx.x, j = tid % LANES, r = blockIdx.y * ROWS + tid / LANES, t0 = blockIdx.x * RUN, t1 = min(t0 + RUN, n_tokens);
    const int C = (nq + nkv) * HD;
    if (rot) {
        for (int i = tid; i < (t1 - t0) * HALF; i += APF_THREADS) {
            float sn, cs;
            sincosf((float)positions[t0 + i / HALF] * inv_freq[i % HALF], &sn, &cs);
            cs_s[i / HALF][i % HALF] = cs * rot_scale;
            sn_s[i / HALF][i % HALF] = sn * rot_scale;
        }
    }
    const bool live = r < nq + nkv, is_k = r >= nq;
    float f[TP][8], w[8];
    const float *nw = is_k ? k_w : q_w;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        const int i = (e >> 2) * HALF + 4 * j + (e & 3);
        w[e] = live && nw ? nw[i] : 1.f;
#pragma unroll
        for (int x = 0; x < TP; ++x) f[x][e] = live && x >= TP - taps ? conv_w[(size_t)(x - (TP - taps)) * C + (size_t)r * HD + i] : 0.f;
    }
    __syncthreads();
    pdl_wait();
    auto go = [&](auto count, int t, int q) {
        constexpr int N = decltype(count)::value;
        const int first = cu_seqlens[q];
        float x[TP - 1 + N][8];
#pragma unroll
        for (int a = 0; a < TP - 1 + N; ++a) {
#pragma unroll
            for (int e = 0; e < 8; ++e) x[a][e] = 0.f;
        }
        const int n0 = t - first - (TP - 1);                  // the first input, among this step's tokens of the request
        auto add = [&](float (&v)[8], const float *src) {
            const float4 lo = *reinterpret_cast<const float4 *>(src), hi = *reinterpret_cast<const float4 *>(src + HALF);
            v[0] += lo.x; v[1] += lo.y; v[2] += lo.z; v[3] += lo.w;
            v[4] += hi.x; v[5] += hi.y; v[6] += hi.z; v[7] += hi.w;
        };
        if (live) {
            const float *src = p + (size_t)t * ld + (size_t)r * HD + 4 * j - (size_t)(TP - 1) * ld;
            for (int s = 0; s < S; ++s, src += slice_stride) {
#pragma unroll
                for (int a = 0; a < TP - 1 + N; ++a)
                    if (a >= TP - taps && n0 + a >= 0 && t + a - (TP - 1) < t1) add(x[a], src + (size_t)a * ld);
            }
            if (n0 < 0) {
                const float *tail = state + (size_t)slots[q] * state_stride + tail_off + (size_t)r * HD + 4 * j;
#pragma unroll
                for (int a = 0; a < TP - 1; ++a)
                    if (a >= TP - taps && n0 + a < 0) add(x[a], tail + (size_t)(taps - 1 + n0 + a) * C);
            }
        }
#pragma unroll
        for (int k = 0; k < N; ++k) {
            float y[8], ss = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                y[e] = 0.f;
#pragma unroll
                for (int a = 0; a < TP; ++a) y[e] = fmaf(f[a][e], x[k + a][e], y[e]);
                ss = fmaf(y[e], y[e], ss);
            }
#pragma unroll
            for (int sh = 1; sh < LANES; sh <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, sh);
            const int tt = t + k;
            if (!live || tt >= t1) continue;
            T *dst;
            if (is_k) {
                const int pos = positions[tt], page = block_table[(size_t)q * table_stride + pos / page_size];
                const size_t slot = (((size_t)page * nkv + (r - nq)) * page_size + pos % page_size) * HD;
                dst = k_cache + slot;
                apf_store4(v_cache + slot + 4 * j, y);
                apf_store4(v_cache + slot + HALF + 4 * j, y + 4);
            } else {
                dst = q_out + ((size_t)tt * nq + r) * HD;
            }
            const float mul = 1.0f / sqrtf(ss / (float)HD + eps);
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] *= mul * w[e];
            if (rot) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float cs = cs_s[tt - t0][4 * j + e], sn = sn_s[tt - t0][4 * j + e], a = y[e], b = y[4 + e];
                    y[e] = a * cs - b * sn;
                    y[4 + e] = b * cs + a * sn;
                }
            }
            apf_store4(dst + 4 * j, y);
            apf_store4(dst + HALF + 4 * j, y + 4);
        }
    };
    const int q0 = seq_of_token[t0];
    if (RUN > 1 && seq_of_token[t1 - 1] == q0) {
        go(ApfCount<RUN>(), t0, q0);
    } else {
        for (int t = t0; t < t1; ++t) go(ApfCount<1>(), t, seq_of_token[t]);
    }
}

template <typename T>
static void apc_launch(dim3 grid, cudaStream_t stream, const float *p, int S, size_t ss, int ld, const float *conv_w, int taps, const float *q_w,
                       const float *k_w, float eps, const float *inv_freq, int rot, float rot_scale, const float *state, size_t st, size_t to,
                       const int *positions, const int *seq_of_token, const int *cu, const int *slots, const int *table, int table_stride, int page_size,
                       T *k_cache, T *v_cache, T *q_out, int n_tokens, int nq, int nkv, int hd, int run) {
    if ((hd == 32 || hd == 64 || hd == 128) && (rot == hd || rot == 0) && taps <= 4 && ld % 4 == 0 && ss % 4 == 0 && st % 4 == 0 && to % 4 == 0 &&
        (((uintptr_t)p | (uintptr_t)state) & 15) == 0) {
        const int per = APF_THREADS / (hd / 8), by = (nq + nkv + per - 1) / per;
#define APF_GO(HD, R) kestrel_launch(attn_prepare_conv_rows_kernel<T, HD, 4, R>, dim3((n_tokens + R - 1) / R, by), dim3(APF_THREADS), 0, stream, p, S, ss, ld, conv_w, taps, \
                                     q_w, k_w, eps, inv_freq, rot, rot_scale, state, st, to, positions, seq_of_token, cu, slots, table, table_stride, page_size, \
                                     k_cache, v_cache, q_out, n_tokens, nq, nkv)
#define APF_HD(HD) { if (run > 1) APF_GO(HD, APC_RUN); else APF_GO(HD, 1); }
        if (hd == 32) APF_HD(32)
        else if (hd == 64) APF_HD(64)
        else APF_HD(128)
#undef APF_HD
#undef APF_GO
        return;
    }
#define APC_GO(PER, TP) kestrel_launch(attn_prepare_conv_kernel<T, PER, TP>, grid, dim3(APC_WARPS * 32), 0, stream, p, S, ss, ld, conv_w, taps, q_w, k_w, eps, \
                                       inv_freq, rot, rot_scale, state, st, to, positions, seq_of_token, cu, slots, table, table_stride, page_size, k_cache, \
                                       v_cache, q_out, n_tokens, nq, nkv, hd, run)
#define APC_TAPS(PER) { if (taps <= 2) APC_GO(PER, 2); else if (taps <= 4) APC_GO(PER, 4); else APC_GO(PER, 9); }
    if (hd <= 64) APC_TAPS(2)
    else if (hd <= 128) APC_TAPS(4)
    else APC_TAPS(8)
#undef APC_TAPS
#undef APC_GO
}

KESTREL_API int kestrel_attn_prepare_conv(const float *partial, int S, long long slice_stride, int ld, const float *conv_w, int taps, const float *q_norm_w,
                                          const float *k_norm_w, float norm_eps, const float *inv_freq, int rot, float rot_scale, float *state,
                                          long long state_stride, long long tail_off, const int *positions, const int *seq_of_token, const int *cu_seqlens,
                                          const int *slots, const int *block_table, int table_stride, int page_size, void *k_cache, void *v_cache,
                                          void *q_out, int dtype, int T, int nseq, int nq, int nkv, int hd, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && nseq > 0 && S > 0 && nq > 0 && nkv > 0 && hd > 0 && hd <= 256 && ld >= (nq + nkv) * hd && page_size > 0, "attn_prepare_conv: bad sizes");
    KESTREL_REQUIRE(taps >= 1 && taps <= 9, "attn_prepare_conv: %d taps, 1 to 9 are built", taps);
    KESTREL_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= hd && (rot == 0 || inv_freq), "attn_prepare_conv: %d rotated dimensions of a head of %d", rot, hd);
    const int run = T >= 512 ? APC_RUN : 1, rows = nq + nkv;
    const dim3 grid((T + run - 1) / run, T >= 512 ? (rows + 4 * APC_WARPS - 1) / (4 * APC_WARPS) : (rows + APC_WARPS - 1) / APC_WARPS);
#define APC_ARGS(TT) grid, stream, partial, S, (size_t)slice_stride, ld, conv_w, taps, q_norm_w, k_norm_w, norm_eps, inv_freq, rot, rot_scale, (const float *)state, \
                     (size_t)state_stride, (size_t)tail_off, positions, seq_of_token, cu_seqlens, slots, block_table, table_stride, page_size, (TT *)k_cache, \
                     (TT *)v_cache, (TT *)q_out, T, nq, nkv, hd, run
    if (dtype == KESTREL_F32) apc_launch<float>(APC_ARGS(float));
    else if (dtype == KESTREL_BF16) apc_launch<__nv_bfloat16>(APC_ARGS(__nv_bfloat16));
    else return kestrel_fail(-2, "attn_prepare_conv: unknown dtype %d", dtype);
#undef APC_ARGS
    int rc = kestrel_check_launch("attn_prepare_conv");
    if (rc) return rc;
    return kestrel_short_conv_tail(partial, S, slice_stride, ld, 0, taps, state, state_stride, tail_off, cu_seqlens, slots, nseq, rows * hd, stream);
}
