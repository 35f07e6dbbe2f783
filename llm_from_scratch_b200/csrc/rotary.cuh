// Rotary angles: products in double precision reduced modulo 2 pi, so a position of any size keeps fp32 accuracy.
#pragma once

#include "common.cuh"

namespace b200 {

// (cos, sin) of position * freq
__device__ __forceinline__ float2 rotary_angle(int64_t position, double freq) {
  double ang = static_cast<double>(position) * freq;
  ang -= 6.283185307179586 * rint(ang * 0.15915494309189535);
  float s, c;
  sincosf(static_cast<float>(ang), &s, &c);
  return make_float2(c, s);
}

}  // namespace b200
