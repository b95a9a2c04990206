// The activations between an expert's two products.
#pragma once
#include "common.cuh"

__device__ __forceinline__ float moe_gelu_erf(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f)); }
// the first product's epilogue: the clamped gated unit of two matrices (MODE 1), the exact gelu of one (MODE 2), or the plain
// silu-gated unit of two (MODE 3)
template <int MODE>
__device__ __forceinline__ float moe_first_act(float a0, float a1, float limit, float alpha);
__device__ __forceinline__ float moe_glu(float g, float u, float limit, float alpha);
template <> __device__ __forceinline__ float moe_first_act<1>(float a0, float a1, float limit, float alpha) { return moe_glu(a0, a1, limit, alpha); }
template <> __device__ __forceinline__ float moe_first_act<2>(float a0, float a1, float limit, float alpha) { return moe_gelu_erf(a0); }
template <> __device__ __forceinline__ float moe_first_act<3>(float a0, float a1, float limit, float alpha) { return silu_f32(a0) * a1; }
template <> __device__ __forceinline__ float moe_first_act<0>(float a0, float a1, float limit, float alpha) { return a0; }
__device__ __forceinline__ float moe_glu(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * (1.0f / (1.0f + expf(-alpha * g))) * (u + 1.0f);
}
