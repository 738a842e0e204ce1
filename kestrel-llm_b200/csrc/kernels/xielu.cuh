// The xIELU activation with two learned numbers p, q and slope 1/2 at zero:
//   z > 0:   softplus(p) z^2 + z / 2
//   z <= 0:  (1/2 + softplus(q)) (exp(z) - 1 - z) + z / 2
#pragma once

__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

struct Xielu {
    float up, down;
    __device__ __forceinline__ Xielu() : up(0.f), down(0.f) {}
    __device__ __forceinline__ explicit Xielu(const float *pq) : up(softplus_f32(pq[0])), down(0.5f + softplus_f32(pq[1])) {}
    __device__ __forceinline__ float operator()(float z) const {
        const float curved = z > 0.f ? up * z * z : down * (expm1f(z) - z);
        return curved + 0.5f * z;
    }
};
