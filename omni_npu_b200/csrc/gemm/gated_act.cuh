// Gated activations that the GEMM epilogues apply to pairs of (gate, up) accumulator columns.
#pragma once

namespace b200 {

enum : int { kActNone = 0, kActSilu = 1, kActClampedGlu = 2 };

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

}  // namespace b200
