// Pieces of the kernels that run a recurrence with a decay per head and token in chunks of 64 tokens on the tensor cores
// (decay_chunks.cu, delta_chunks.cu).
#pragma once
#include "common.cuh"
#include "mma_sync.cuh"

#define DC_C 64                  // tokens of a chunk
#define DC_N 64                  // value columns worked on at a time
#define DC_LDN (DC_N + 8)        // row lengths in shared memory that keep ldmatrix free of bank conflicts

// two bfloat16 terms of a float32: the rounded value and what it leaves, 16 bits of mantissa together
__device__ __forceinline__ void dc_split(float x, __nv_bfloat16 &hi, __nv_bfloat16 &lo) {
    hi = __float2bfloat16_rn(x);
    lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}
__device__ __forceinline__ uint32_t dc_bits(__nv_bfloat16 a, __nv_bfloat16 b) {
    __nv_bfloat162 v;
    v.x = a;
    v.y = b;
    return *reinterpret_cast<uint32_t *>(&v);
}
// both terms of two neighbours, packed
__device__ __forceinline__ void dc_split2(float x, float y, uint32_t &hi, uint32_t &lo) {
    __nv_bfloat16 a, b, c, d;
    dc_split(x, a, c);
    dc_split(y, b, d);
    hi = dc_bits(a, b);
    lo = dc_bits(c, d);
}
__device__ __forceinline__ uint32_t dc_smem(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void dc_cp16(__nv_bfloat16 *dst, const __nv_bfloat16 *src, bool valid) {
    const int sz = valid ? 16 : 0;                    // 0: sixteen zero bytes
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dc_smem(dst)), "l"(src), "r"(sz) : "memory");
}
__device__ __forceinline__ void dc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void dc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// n rows of d numbers (of DC_C, of D) into shared memory [DC_C][D + 8], zero beyond them; THREADS threads
template <int D, int THREADS = 128>
__device__ __forceinline__ void dc_load_rows(__nv_bfloat16 *dst, const __nv_bfloat16 *src, size_t row_stride, int n, int d, int tid) {
    for (int idx = tid; idx < DC_C * (D / 8); idx += THREADS) {
        const int r = idx / (D / 8), c = idx % (D / 8) * 8;
        const bool ok = r < n && c < d;
        dc_cp16(dst + r * (D + 8) + c, src + (ok ? (size_t)r * row_stride + c : 0), ok);
    }
}

// The running sums of a chunk's logarithms of decays, by the first warp: sums[i] = log of the decay from in front of the chunk to
// behind its token i; tokens beyond n add nothing.
__device__ __forceinline__ void dc_running_sums(float *sums, const float *log_decay, size_t stride, int n, int tid) {
    if (tid < 32) {
        const float a = 2 * tid < n ? log_decay[(size_t)(2 * tid) * stride] : 0.f;
        const float b = 2 * tid + 1 < n ? log_decay[(size_t)(2 * tid + 1) * stride] : 0.f;
        float s = a + b;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(0xffffffffu, s, o);
            if (tid >= o) s += x;
        }
        sums[2 * tid] = s - b;
        sums[2 * tid + 1] = s;
    }
}
