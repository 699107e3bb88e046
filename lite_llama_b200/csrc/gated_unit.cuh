// Gated activation units shared by the element-wise kernels and the grouped products' epilogues (fp32 arithmetic):
//   kUnitSilu      silu(g) * u
//   kUnitGeluTanh  gelu(g) * u, tanh form
//   kUnitClamped   g' = min(g, limit), u' = clamp(u, -limit, limit):   g' * sigmoid(alpha g') * (u' + 1)
#pragma once
#include "common.cuh"

constexpr int kUnitSilu = 0, kUnitClamped = 1, kUnitGeluTanh = 2;

struct GatedUnit {
  int form;
  float limit, alpha;
  __device__ __forceinline__ float operator()(float g, float u) const {
    if (form == kUnitClamped) {
      g = fminf(g, limit);
      u = fminf(fmaxf(u, -limit), limit);
      return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
    }
    if (form == kUnitGeluTanh) return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
    return g / (1.0f + expf(-g)) * u;
  }
};
