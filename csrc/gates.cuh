// Activations of two operands, shared by the products' epilogues and by the kernel that takes them alone.
#pragma once
#include <cuda_runtime.h>

namespace tyr {

// Clamped SwiGLU: g = min(gate, limit), u = clamp(up, -limit, limit); g sigmoid(slope g) (u + 1).
__device__ __forceinline__ float clamped_swiglu(float gate, float up, float limit, float slope) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-slope * g)) * (u + 1.f);
}

// tanh-GELU, as z sigmoid(2 a) with a the argument of the tanh.
__device__ __forceinline__ float gelu_tanh(float z) {
  return z / (1.f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}

}  // namespace tyr
