// The gated activations of feed-forwards, float32 arithmetic.
#pragma once

#include "common.cuh"

__device__ __forceinline__ float silu_mul(float g, float u) { return g / (1.0f + expf(-g)) * u; }
// For results that are rounded to bfloat16: the hardware exponential and reciprocal (errors of
// a few 1e-7 relative, a thousand times below the rounding), a third of the instructions
// (42.4 against 47.8 us for 2,048 tokens of the 7B shape).
__device__ __forceinline__ float silu_mul_fast(float g, float u) {
    return g * __frcp_rn(1.0f + __expf(-g)) * u;
}

// the tanh form of GELU: 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3)))
__device__ __forceinline__ float gelu_tanh_mul(float g, float u) {
    return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
}
// the clamped form: g = min(gate, limit), u = clamp(up, -limit, limit), g sigmoid(alpha g) (u + 1)
__device__ __forceinline__ float swish_clamped_mul(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
}
// ACT 0: SiLU; 1: GELU (tanh form); 2: the clamped form with p0 = limit, p1 = alpha
template <int ACT> __device__ __forceinline__ float act_mul(float g, float u, float p0, float p1) {
    return ACT == 2 ? swish_clamped_mul(g, u, p0, p1) : ACT == 1 ? gelu_tanh_mul(g, u) : silu_mul(g, u);
}
template <int ACT> __device__ __forceinline__ float act_mul_fast(float g, float u, float p0, float p1) {
    return ACT == 2 ? swish_clamped_mul(g, u, p0, p1) : ACT == 1 ? gelu_tanh_mul(g, u) : silu_mul_fast(g, u);
}
// the same with the form as an argument
__device__ __forceinline__ float act_mul_of(int act, float g, float u, float p0, float p1) {
    return act == 2 ? swish_clamped_mul(g, u, p0, p1) : act == 1 ? gelu_tanh_mul(g, u) : silu_mul(g, u);
}
