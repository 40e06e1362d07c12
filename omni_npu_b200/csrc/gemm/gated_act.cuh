// Activations of the GEMM epilogues: gated ones on pairs of (gate, up) accumulator columns, and one on
// single columns.
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

namespace b200 {

enum : int { kActNone = 0, kActSilu = 1, kActClampedGlu = 2, kActXielu = 3, kActGeluTanh = 4, kActRelu2 = 5, kActTanh = 6,
             kActReluGate = 7 };

//   kActSilu        silu(g) * u
//   kActClampedGlu  g' * sigmoid(alpha * g') * (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit)
//   kActGeluTanh    g / 2 * (1 + tanh(z)) * u = g * sigmoid(2 z) * u with z = sqrt(2 / pi) (g + 0.044715 g^3)
//   kActReluGate    max(g, 0) * u
__device__ __forceinline__ float gelu_exponent(float g) {
  return -1.5957691216057308f * fmaf(0.044715f * g * g, g, g);       // -2 z
}
__device__ __forceinline__ float gated_act(int kind, float g, float u, float alpha, float limit) {
  if (kind == kActClampedGlu) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + __expf(-alpha * g)) * (u + 1.f);
  }
  if (kind == kActReluGate) return fmaxf(g, 0.f) * u;
  return g / (1.f + __expf(kind == kActGeluTanh ? gelu_exponent(g) : -g)) * u;
}
// the same with the exact fp32 functions, for products that are not rounded to bf16
__device__ __forceinline__ float gated_act_exact(int kind, float g, float u, float alpha, float limit) {
  if (kind == kActClampedGlu) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-alpha * g)) * (u + 1.f);
  }
  if (kind == kActReluGate) return fmaxf(g, 0.f) * u;
  return g / (1.f + expf(kind == kActGeluTanh ? gelu_exponent(g) : -g)) * u;
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

// Activations of single columns:
//   kActRelu2       max(z, 0)^2
//   kActTanh        tanh(z) = 1 - 2 / (exp(2 z) + 1) (absolute error 2e-7)
__device__ __forceinline__ float unary_act(int kind, float z, float alpha, float limit) {
  if (kind == kActRelu2) {
    z = fmaxf(z, 0.f);
    return z * z;
  }
  if (kind == kActTanh) return 1.f - 2.f / (__expf(2.f * fminf(z, 40.f)) + 1.f);
  return xielu(z, alpha, limit);
}
__device__ __forceinline__ float unary_act_exact(int kind, float z, float alpha, float limit) {
  if (kind == kActRelu2) {
    z = fmaxf(z, 0.f);
    return z * z;
  }
  return kind == kActTanh ? tanhf(z) : xielu_exact(z, alpha, limit);
}

// v[i] += bias[col + i] for the columns below N.  Whole, aligned groups are two 16-byte loads, the same address
// in every lane.
__device__ __forceinline__ void add_bias16(float (&v)[16], const __nv_bfloat16* bias, int col, int N) {
  const __nv_bfloat16* b = bias + col;
  if (col + 16 <= N && (reinterpret_cast<uintptr_t>(b) & 15) == 0) {
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const uint4 u = __ldg(reinterpret_cast<const uint4*>(b) + h);
      const uint32_t r[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[8 * h + 2 * i] += __uint_as_float(r[i] << 16);
        v[8 * h + 2 * i + 1] += __uint_as_float(r[i] & 0xffff0000u);
      }
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < 16; ++i)
    if (col + i < N) v[i] += __bfloat162float(b[i]);
}

// Whether a kind joins pairs of columns (half as many come out), or works on single ones.
__host__ __device__ __forceinline__ bool act_is_gated(int kind) {
  return kind == kActSilu || kind == kActClampedGlu || kind == kActGeluTanh || kind == kActReluGate;
}
__host__ __device__ __forceinline__ bool act_is_unary(int kind) {
  return kind == kActXielu || kind == kActRelu2 || kind == kActTanh;
}

}  // namespace b200
