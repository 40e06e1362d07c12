// Activations of the GEMM epilogues: gated ones on pairs of (gate, up) accumulator columns, and one on
// single columns.
#pragma once

namespace b200 {

enum : int { kActNone = 0, kActSilu = 1, kActClampedGlu = 2, kActXielu = 3 };

//   kActSilu        silu(g) * u
//   kActClampedGlu  g' * sigmoid(alpha * g') * (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit)
__device__ __forceinline__ float gated_act(int kind, float g, float u, float alpha, float limit) {
  if (kind == kActClampedGlu) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + __expf(-alpha * g)) * (u + 1.f);
  }
  return (g / (1.f + __expf(-g))) * u;
}

//   kActXielu       z > 0: alpha * z^2 + z / 2;  z <= 0: limit * (exp(z) - 1 - z) + z / 2
// (results rounded to bf16: near zero the absolute error of the difference, 2e-7, is below half a step of
// z / 2 wherever that exceeds 1e-4)
__device__ __forceinline__ float xielu(float z, float alpha, float limit) {
  const float a = z > 0.f ? alpha * z * z : limit * (__expf(z) - 1.f - z);
  return fmaf(0.5f, z, a);
}
__device__ __forceinline__ float xielu_exact(float z, float alpha, float limit) {
  const float a = z > 0.f ? alpha * z * z : limit * (expm1f(z) - z);
  return fmaf(0.5f, z, a);
}

// Whether a kind joins pairs of columns (half as many come out).
__host__ __device__ __forceinline__ bool act_is_gated(int kind) { return kind == kActSilu || kind == kActClampedGlu; }

}  // namespace b200
