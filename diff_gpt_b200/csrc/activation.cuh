// Activations that more than one kernel applies (element-wise launches and GEMM epilogues).
#pragma once

namespace dgpt {

// z > 0:   alpha_p z^2 + z / 2
// z <= 0:  alpha_n (e^z - 1 - z) + z / 2
// alpha_p = softplus(p) and alpha_n = 1/2 + softplus(q) of the layer's two learned numbers.
__device__ __forceinline__ float xielu_value(float z, float alpha_p, float alpha_n) {
  const float curve = z > 0.f ? alpha_p * z * z : alpha_n * (expm1f(z) - z);
  return fmaf(0.5f, z, curve);
}

// The same for a result that is rounded to bf16: e^z from the exponential unit, with an absolute error near 1e-7 (below
// a bf16 step of the sum wherever that is larger than 1e-4), a third of the instructions.
__device__ __forceinline__ float xielu_fast(float z, float alpha_p, float alpha_n) {
  const bool pos = z > 0.f;
  const float t = pos ? z * z : __expf(z) - 1.f - z;
  return fmaf(pos ? alpha_p : alpha_n, t, 0.5f * z);
}

// gate * sigmoid(gate) * up
__device__ __forceinline__ float silu_mul_value(float gate, float up) { return gate / (1.f + expf(-gate)) * up; }
// The same for a result that is rounded to bf16 (fast exponential and division, relative error near 1e-6).
__device__ __forceinline__ float silu_mul_fast(float gate, float up) { return __fdividef(gate, 1.f + __expf(-gate)) * up; }

}  // namespace dgpt
