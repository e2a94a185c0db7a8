// The angle of a rotary position and its cosine and sine.
#pragma once

#include "common.cuh"

namespace le {

// (cosine, sine) of position * rate, times `magnitude`: the angle is taken in 64 bits and brought into [-pi, pi] there
// (a 32-bit product would be off by up to position * 2^-24 radians), its cosine and sine are 32-bit.
__device__ __forceinline__ float2 turn_of(int position, double rate, float magnitude) {
  double a = static_cast<double>(position) * rate;
  a -= 6.283185307179586 * rint(a * 0.15915494309189535);
  float s, c;
  sincosf(static_cast<float>(a), &s, &c);
  return make_float2(c * magnitude, s * magnitude);
}

// Rates in either width: float64 ones as above; float32 ones give the angle position * rate in 32 bits.
struct Rates {
  const void *data;
  int wide;           // 1: float64, 0: float32
};
__device__ __forceinline__ float2 turn_of(int position, const Rates &rates, int i, float magnitude) {
  if (rates.wide) return turn_of(position, static_cast<const double *>(rates.data)[i], magnitude);
  float s, c;
  sincosf(static_cast<float>(position) * static_cast<const float *>(rates.data)[i], &s, &c);
  return make_float2(c * magnitude, s * magnitude);
}

// Neighbouring entries (u, v) turned.
__device__ __forceinline__ void turn_pair(float &u, float &v, const float2 &cs) {
  const float nu = u * cs.x - v * cs.y, nv = v * cs.x + u * cs.y;
  u = nu, v = nv;
}

}  // namespace le
