// Rotation angles that lose nothing at far positions.
#pragma once

namespace dgpp {

// sin and cos of pos * f_i.  freq [2, half]: f as a leading and a residual term; the rounding error of the fp32 product and the
// residual turn the result by a small angle.
__device__ __forceinline__ void rope_angle(const float* freq, int half, int pos, int i, float& s, float& c) {
  const float p = static_cast<float>(pos), hi = freq[i], ang = p * hi;
  const float err = fmaf(p, hi, -ang) + p * freq[half + i];
  float s0, c0;
  sincosf(ang, &s0, &c0);
  s = fmaf(c0, err, s0);
  c = fmaf(-s0, err, c0);
}

}  // namespace dgpp
