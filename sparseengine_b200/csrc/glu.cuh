// The gated activations an expert's first product ends in.  `gate` and `up` arrive rounded to the
// activation type T; the result is 32-bit and the caller rounds it once more as it stores it.
//   kind 0  silu(gate) * up, silu rounded to T before the product (the rounding points of the
//           bfloat16 pipeline the other kernels keep)
//   kind 1  g = min(gate, limit), u = clamp(up, -limit, limit): g * sigmoid(alpha * g) * (u + 1)
//   kind 2  gelu(gate) * up, gelu in its tanh form
#pragma once
#include "common.cuh"

#define SE_GLU_SILU 0
#define SE_GLU_CLAMPED 1
#define SE_GLU_GELU 2

namespace se {

// 0.5 z (1 + tanh(u)) = z sigmoid(2u) with u = sqrt(2/pi) (z + 0.044715 z^3).  Results that are rounded to 16 bits
// next take the fast exponential and quotient; 32-bit ones tanhf.
template <typename T>
__device__ __forceinline__ float gelu_tanh(float z) {
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    if (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-2.f * u));
    return 0.5f * z * (1.f + tanhf(u));
}

template <typename T>
__device__ __forceinline__ float glu_value(float gate, float up, int kind, float limit, float alpha) {
    if (kind == SE_GLU_CLAMPED) {
        const float g = fminf(gate, limit);
        const float u = fminf(fmaxf(up, -limit), limit);
        return g / (1.f + expf(-alpha * g)) * (u + 1.f);
    }
    if (kind == SE_GLU_GELU) return gelu_tanh<T>(gate) * up;
    return round_act<T>(gate / (1.f + expf(-gate))) * up;
}

}  // namespace se
