// A sub-layer's output on its way into the 32-bit residual stream ("addend"):
// [rows, W] in the activations' type, or float32 partial sums [parts, rows, W]
// of a split-K product, which are added in order; and accesses to four
// neighbouring values at once.
#pragma once

#include "common.cuh"

namespace le {

struct Addend {
  const void *data;     // null: none
  int dtype;
  int parts;
  int64_t part_stride;  // elements between partial sums
};

__device__ __forceinline__ float addend_at(const Addend &a, int64_t at) {
  if (a.dtype == LE_BF16) return to_f32(static_cast<const __nv_bfloat16 *>(a.data)[at]);
  const float *p = static_cast<const float *>(a.data);
  float v = p[at];
  for (int s = 1; s < a.parts; ++s) v += p[at + s * a.part_stride];
  return v;
}

// Four consecutive values at once (the address a multiple of 16 bytes for floats, of 8 for bfloat16).
__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16 *p) {
  const uint2 r = *reinterpret_cast<const uint2 *>(p);
  return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xffff0000u), __uint_as_float(r.y << 16),
                     __uint_as_float(r.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16 *p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 r;
  r.x = *reinterpret_cast<const uint32_t *>(&lo), r.y = *reinterpret_cast<const uint32_t *>(&hi);
  *reinterpret_cast<uint2 *>(p) = r;
}
__device__ __forceinline__ float4 addend4(const Addend &a, int64_t at) {
  if (a.dtype == LE_BF16) return load4(static_cast<const __nv_bfloat16 *>(a.data) + at);
  const float *p = static_cast<const float *>(a.data);
  float4 v = load4(p + at);
  for (int s = 1; s < a.parts; ++s) {
    const float4 w = load4(p + at + s * a.part_stride);
    v.x += w.x, v.y += w.y, v.z += w.z, v.w += w.w;
  }
  return v;
}

inline bool on16(const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

}  // namespace le
