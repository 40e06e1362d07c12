// What the recurrent layers' kernels share: activations in full fp32 accuracy (their sources are compiled
// without the fast-math flag).
#pragma once

#include <cuda_runtime.h>

namespace b200 {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

}  // namespace b200
