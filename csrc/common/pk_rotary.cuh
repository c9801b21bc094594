// Rotary positions: angle = position x frequency in double precision, reduced by whole turns, sine and cosine in fp32.
#pragma once
#include "pk_common.cuh"

namespace pk {

__device__ __forceinline__ void rotary_sincos(double freq, int pos, float& s, float& c) {
  double a = (double)pos * freq;
  a -= 6.283185307179586476925286766559 * rint(a * 0.15915494309189533576888376337251);
  sincosf((float)a, &s, &c);
}

// (u, v) turned by the angle: u cos - v sin, v cos + u sin
__device__ __forceinline__ void rotate_pair(float& u, float& v, float s, float c) {
  const float a = u * c - v * s, b = v * c + u * s;
  u = a;
  v = b;
}

}  // namespace pk
