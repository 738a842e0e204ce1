// The activation between a gated feed-forward's two halves, from a gate g and an up value u:
//   limit <= 0   silu(g) u
//   limit > 0    both bounded first, g <- min(g, limit), u <- clamp(u, -limit, limit), then g sigmoid(1.702 g) (u + 1)
#pragma once

#define GATED_CLAMP_SLOPE 1.702f

__device__ __forceinline__ float gated_act(float g, float u, float limit) {
    if (limit > 0.f) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g / (1.0f + expf(-GATED_CLAMP_SLOPE * g)) * (u + 1.0f);
    }
    return g / (1.0f + expf(-g)) * u;
}
// the same on the 2-ulp float32 intrinsics, for results that are rounded to bfloat16
__device__ __forceinline__ float gated_act_fast(float g, float u, float limit) {
    if (limit > 0.f) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return __fdividef(g, 1.0f + __expf(-GATED_CLAMP_SLOPE * g)) * (u + 1.0f);
    }
    return __fdividef(g, 1.0f + __expf(-g)) * u;
}
