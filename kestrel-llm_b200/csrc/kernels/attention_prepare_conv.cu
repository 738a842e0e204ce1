// The step between a fused query/key product and attention, for mixers whose queries and keys pass a short causal convolution and
// whose values ARE their keys:
//
//   u[t, c] = sum_j w[c, j] x[t - (taps - 1) + j, c]        per column of [q: nq hd | k: nkv hd]; inputs before a request's first
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
            for (int j = 0; j < TP; ++j) f[j][c] = i < hd && j >= TP - taps ? conv_w[((size_t)r * hd + i) * taps + j - (TP - taps)] : 0.f;
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

template <typename T>
static void apc_launch(dim3 grid, cudaStream_t stream, const float *p, int S, size_t ss, int ld, const float *conv_w, int taps, const float *q_w,
                       const float *k_w, float eps, const float *inv_freq, int rot, float rot_scale, const float *state, size_t st, size_t to,
                       const int *positions, const int *seq_of_token, const int *cu, const int *slots, const int *table, int table_stride, int page_size,
                       T *k_cache, T *v_cache, T *q_out, int n_tokens, int nq, int nkv, int hd, int run) {
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
