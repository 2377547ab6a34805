// Activations by number, shared by the kernels around gated mixers and feed-forwards:
// 0 none, 1 sigmoid, 2 silu, 3 gelu (tanh form), 4 the square of relu, 5 the clamped form (its kernels spell it out), 6 relu.
#pragma once
#include "common.cuh"

__device__ __forceinline__ float go_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float go_gelu_tanh(float v) {
    return 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
}
__device__ __forceinline__ float go_act(float v, int act) {
    return act == 1 ? go_sigmoid(v) : act == 2 ? v * go_sigmoid(v) : act == 3 ? go_gelu_tanh(v) : act == 4 ? (v > 0.f ? v * v : 0.f)
         : act == 6 ? fmaxf(v, 0.f) : v;
}

// For results that are rounded to bfloat16: sigmoid and tanh from the special-function unit's 2^x and reciprocal (relative
// error about 2^-22, far below that rounding).
__device__ __forceinline__ float go_sigmoid_fast(float v) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-1.4426950408889634f * v));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
    return r;
}
__device__ __forceinline__ float go_act_fast(float v, int act) {
    if (act == 2) return v * go_sigmoid_fast(v);
    if (act == 3) return v * go_sigmoid_fast(1.5957691216057308f * (v + 0.044715f * v * v * v));   // 0.5 v (1 + tanh(u)) = v sigmoid(2u)
    if (act == 1) return go_sigmoid_fast(v);
    if (act == 6) return fmaxf(v, 0.f);
    return v;
}
