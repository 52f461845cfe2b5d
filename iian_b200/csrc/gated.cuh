// The activation between a gated feed-forward's two matrices, shared by the kernels that apply it: on their own rows, in a
// product's epilogue, between the grouped products of routed experts.
#pragma once

namespace iian {

// codes of the activations; ACT_RELU2 belongs to feed-forwards without a gate and has no value here
enum { ACT_SILU = 0, ACT_GELU_TANH = 1, ACT_CLAMPED = 2, ACT_RELU2 = 3, ACT_RELU = 4 };

// silu(g) u;  gelu_tanh(g) u;  max(g, 0) u;  clamped: with g' = min(g, limit), u' = clamp(u, -limit, limit):
// g' sigmoid(1.702 g') (u' + 1)
__device__ __forceinline__ float gated_value(float g, float u, int act, float limit) {
    if (act == ACT_SILU) return g / (1.0f + expf(-g)) * u;
    if (act == ACT_RELU) return fmaxf(g, 0.0f) * u;
    if (act == ACT_CLAMPED) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
    }
    const float t = 0.7978845608028654f * (g + 0.044715f * g * g * g);
    return 0.5f * g * (1.0f + tanhf(t)) * u;
}

// the same with the hardware's exponential, for results that are rounded to bfloat16 next
__device__ __forceinline__ float gated_value_fast(float g, float u, int act, float limit) {
    if (act == ACT_SILU) return g / (1.0f + __expf(-g)) * u;
    if (act == ACT_RELU) return fmaxf(g, 0.0f) * u;
    g = fminf(g, limit);                                     // ACT_CLAMPED
    u = fminf(fmaxf(u, -limit), limit);
    return __fdividef(g, 1.0f + __expf(-1.702f * g)) * (u + 1.0f);
}

}  // namespace iian
