// Single-instruction approximations (about 2^-22 relative, denormals flushed) for kernels that name them, and the soft cap of
// attention scores, cap * tanh(s / cap), on them.
#pragma once

namespace b200 {

__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// A raw score s becomes out * tanh(scale * s / cap).
struct SoftCap {
  float in2;    // 2 log2(e) scale / cap: one multiplication makes the exponent of e^(2 x)
  float out;    // cap (times log2(e) where scores are in log2 units)
};
// tanh(x) = 1 - 2 / (1 + e^(2 x)): the error is a few 2^-23 of the cap at every x, e^(2 x) may overflow or vanish.
__device__ __forceinline__ float soft_cap(float s, const SoftCap& c) {
  return fmaf(-2.f * c.out, rcp_approx(1.f + ex2_approx(s * c.in2)), c.out);
}

}  // namespace b200
