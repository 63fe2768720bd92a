// The activations of feed-forwards without a gate, by the numbers that the entry points take:
// 0 relu(x)^2; 1 gelu in its tanh form; 2 silu; 3 gelu in its exact form, x Phi(x); and the clamped gate
// g' sigmoid(1.702 g') (u' + 1), g' = min(g, limit), u' = clamp(u, -limit, limit).
#pragma once
#include <math.h>

constexpr int FMX_ACTS = 4;

__device__ __forceinline__ float act_f(int kind, float x) {
  if (kind == 0) { const float p = fmaxf(x, 0.f); return p * p; }
  if (kind == 1) return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
  if (kind == 3) return 0.5f * x * (1.0f + erff(x * 0.7071067811865476f));
  return x / (1.0f + expf(-x));
}

__device__ __forceinline__ float clamped_gate(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return (g / (1.0f + expf(-1.702f * g))) * (u + 1.0f);
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
