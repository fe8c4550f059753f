// Activations shared by row kernels and GEMM epilogues.
#pragma once

#include "common.cuh"

namespace b200 {

// xIELU with its two learned numbers already mapped to curvatures: z > 0: pos z^2 + z / 2;
// z <= 0: neg (e^z - 1 - z) + z / 2   (pos = softplus(p), neg = 1/2 + softplus(q))
__device__ __forceinline__ float xielu_exact(float z, float pos, float neg) {
  const float zn = fminf(z, 0.f);
  return z > 0.f ? fmaf(pos * z, z, 0.5f * z) : fmaf(neg, expm1f(zn) - zn, 0.5f * z);
}

// The same for results that are rounded to 16 bits: e^z - 1 - z by its power series near 0, where the
// difference would cancel, and by the hardware exponential elsewhere (relative error below 1e-5).
__device__ __forceinline__ float xielu_fast(float z, float pos, float neg) {
  const float zn = fminf(z, 0.f);
  const float e = fast_exp2(zn * 1.4426950408889634f) - 1.0f - zn;
  float s = fmaf(zn, 1.0f / 720.0f, 1.0f / 120.0f);
  s = fmaf(zn, s, 1.0f / 24.0f);
  s = fmaf(zn, s, 1.0f / 6.0f);
  s = fmaf(zn, s, 0.5f) * zn * zn;
  const float n = zn > -0.25f ? s : e;
  return fmaf(z > 0.f ? pos * z : 0.f, z, fmaf(neg, n, 0.5f * z));
}

}  // namespace b200
