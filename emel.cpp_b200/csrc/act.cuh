// Scalar activations of layered decoders, f32.
#pragma once

#include <cuda_runtime.h>
#include <math.h>

namespace emelb {

__device__ __forceinline__ float sigmoidf_(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float siluf_(float z) { return z / (1.0f + expf(-z)); }
// 0.5 z (1 + tanh(y)) = z sigmoid(2 y), y = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanhf_(float z) {
  return z / (1.0f + expf(-1.5957691216057308f * fmaf(0.044715f * z * z, z, z)));
}
__device__ __forceinline__ float softplusf_(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
// cap tanh(z / cap); cap 0: z
__device__ __forceinline__ float softcapf_(float z, float cap) { return cap > 0.0f ? cap * tanhf(z / cap) : z; }

}  // namespace emelb
