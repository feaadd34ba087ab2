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

}  // namespace dgpt
