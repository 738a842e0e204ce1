// Retention: linear attention with a fixed decay per head.  Per head, with d key and dv value channels,
//
//   S_t = decay S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t
//
// q and k rotated by position (rotate-half pairs of a head's first `rot` dimensions), k times d^-1/2 afterwards.  S is float32,
// [d, dv] a head, in the request's state slot.
#include "common.cuh"
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

KESTREL_API int kestrel_retention_prepare(const float *partial, int S, long long slice_stride, int ld, const int *positions, const float *inv_freq,
                                          int rot, const float *decay, void *q_out, void *k_out, void *v_out, float *w_out, int dtype, int T, int H,
                                          int d, int dv, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && S > 0 && H > 0 && d > 0 && dv > 0 && ld >= H * (2 * d + dv), "retention_prepare: bad sizes");
    KESTREL_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= d && (rot == 0 || inv_freq), "retention_prepare: %d rotated dimensions of a head of %d", rot, d);
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
