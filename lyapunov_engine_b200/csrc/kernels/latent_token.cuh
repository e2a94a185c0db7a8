// One token's part in latent attention, as a block's work for kernels that run
// it alone or beside other work: its latent's norm, its rotated key part's turn
// and their cache write; and the turns of its queries' rotated parts on their
// way behind the queries in the latent space.
#pragma once

#include "turn.cuh"

namespace le_latent {

constexpr int MAX_PAIRS = 256;      // rotated parts of up to 512 entries

template <typename T>
struct Args {
  const T *src;                     // the projection's rows
  int64_t src_stride;
  int col, rank, rot, padded;       // the latent at columns [col, col + rank), its rotated part in the rot columns behind it
  const float *weight;              // [rank]
  float eps;
  le::Rates rates;                  // [rot / 2]
  float magnitude;                  // on cosines and sines
  T *cache;                         // [pages, 1, page, padded] or null: nothing is stored
  const int32_t *positions, *request_of_token, *block_table;
  int max_blocks, page_size, num_pages;
  int *status;
  // queries: head h's rotated entries at columns q_col + h * q_head of the row, turned to columns h * padded + rank ..
  // of q_out's row, zeros up to (h + 1) * padded; q_out null: none
  int q_col, q_head, heads;
  T *q_out;
  int64_t q_stride;
  int q_pairs;                      // rows and columns are such that two neighbours are one access
};

// Needs no result of the kernel before this one.
template <typename T>
__device__ __forceinline__ void make_turns(float2 *turn, const Args<T> &a, int t) {
  for (int i = threadIdx.x; i < (a.rot >> 1); i += blockDim.x) turn[i] = le::turn_of(a.positions[t], a.rates, i, a.magnitude);
}

// The whole block; `turn` is made, `scratch` holds 33 floats.
template <typename T>
__device__ __forceinline__ void store_latent(const Args<T> &a, int t, const float2 *turn, float *scratch) {
  const int pos = a.positions[t];
  const int b = a.request_of_token[t];
  const int page = pos >= 0 ? a.block_table[static_cast<int64_t>(b) * a.max_blocks + pos / a.page_size] : -1;
  const bool bad = page < 0 || page >= a.num_pages;
  if (bad && threadIdx.x == 0) atomicOr(a.status, LE_STATUS_BAD_PAGE);
  const T *x = a.src + static_cast<int64_t>(t) * a.src_stride + a.col;
  float ss = 0.0f;
  for (int i = threadIdx.x; i < a.rank; i += blockDim.x) {
    const float v = le::to_f32(x[i]);
    ss = fmaf(v, v, ss);
  }
  ss = le::block_sum(ss, scratch);
  if (bad) return;
  const float inv = rsqrtf(ss / static_cast<float>(a.rank) + a.eps);
  T *dst = a.cache + (static_cast<int64_t>(page) * a.page_size + pos % a.page_size) * a.padded;
  for (int i = threadIdx.x; i < a.padded; i += blockDim.x) {
    float v = 0.0f;
    if (i < a.rank) {
      v = le::to_f32(x[i]) * inv * a.weight[i];
    } else if (i < a.rank + a.rot) {
      const int j = i - a.rank;
      v = le::to_f32(x[i]);
      const float other = le::to_f32(x[a.rank + (j ^ 1)]);
      const float2 cs = turn[j >> 1];
      v = (j & 1) ? v * cs.x + other * cs.y : v * cs.x - other * cs.y;
    }
    dst[i] = le::from_f32<T>(v);
  }
}

// The whole block, block `mine` of `blocks` that share the token's work; `turn` is made.
template <typename T>
__device__ __forceinline__ void turn_queries(const Args<T> &a, int t, const float2 *turn, int mine = 0, int blocks = 1) {
  const T *row = a.src + static_cast<int64_t>(t) * a.src_stride + a.q_col;
  T *out = a.q_out + static_cast<int64_t>(t) * a.q_stride + a.rank;
  const int half = a.rot >> 1, tail = a.padded - a.rank - a.rot;
  const int first = mine * blockDim.x + threadIdx.x, step = blocks * blockDim.x;
  for (int i = first; i < a.heads * half; i += step) {
    const int h = i / half, j = i - h * half;
    const T *p = row + static_cast<int64_t>(h) * a.q_head + 2 * j;
    T *o = out + static_cast<int64_t>(h) * a.padded + 2 * j;
    if (a.q_pairs) {
      if constexpr (sizeof(T) == 2) {
        const uint32_t r = *reinterpret_cast<const uint32_t *>(p);
        float u = __uint_as_float(r << 16), v = __uint_as_float(r & 0xffff0000u);
        le::turn_pair(u, v, turn[j]);
        *reinterpret_cast<__nv_bfloat162 *>(o) = __floats2bfloat162_rn(u, v);
      } else {
        float2 r = *reinterpret_cast<const float2 *>(p);
        le::turn_pair(r.x, r.y, turn[j]);
        *reinterpret_cast<float2 *>(o) = r;
      }
    } else {
      float u = le::to_f32(p[0]), v = le::to_f32(p[1]);
      le::turn_pair(u, v, turn[j]);
      o[0] = le::from_f32<T>(u), o[1] = le::from_f32<T>(v);
    }
  }
  for (int i = first; i < a.heads * tail; i += step)
    out[static_cast<int64_t>(i / tail) * a.padded + a.rot + i % tail] = le::from_f32<T>(0.0f);
}

template <typename T>
inline int pairs_together(const Args<T> &a) {
  return a.src_stride % 2 == 0 && a.q_col % 2 == 0 && a.q_head % 2 == 0 && a.q_stride % 2 == 0 && a.rank % 2 == 0 &&
         a.padded % 2 == 0 && reinterpret_cast<uintptr_t>(a.src) % (2 * sizeof(T)) == 0 &&
         reinterpret_cast<uintptr_t>(a.q_out) % (2 * sizeof(T)) == 0;
}

}  // namespace le_latent
