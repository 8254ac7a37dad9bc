// Rotation angles, all in 32-bit.  A pair's speed is given in turns per position as two floats (value and remainder), so the
// fraction of a turn is as exact at position 10^6 as at position 1.
#pragma once
#include <cuda_runtime.h>

namespace gk {

__device__ __forceinline__ void rotation_at(int pos, float2 turns, float* sin_out, float* cos_out) {
  const float x = static_cast<float>(pos), t = x * turns.x;
  const float frac = (t - rintf(t)) + fmaf(x, turns.y, fmaf(x, turns.x, -t));
  sincospif(2.f * frac, sin_out, cos_out);
}

}  // namespace gk
