// The few-rows form of the per-head products (see gemm_heads.cu) as a block's
// work, for kernels that run it beside other work in one launch.
#pragma once

#include "common.cuh"

namespace le_heads {

constexpr int GR_ROWS = 8;      // rows of a a block takes (blockIdx.z walks the rest)
constexpr int GR_COLS = 4;      // output columns per warp
constexpr int GR_WARPS = 4;

// Where the heads lie in a row and what gates them.
struct Heads {
  int64_t a_head, out_head;     // elements between two heads of a row of a / of out (at least K / N)
  int gate_entries;             // the gate has a number per head (0) or per entry: head h's at columns h * N ..
};

// The work of one block of the few-rows form (blockIdx.x: 16 output columns, blockIdx.y: the head, blockIdx.z: 8 rows).
template <typename T>
__device__ __forceinline__ void gemm_heads_rows_block(T *__restrict__ out, int64_t out_stride, const T *__restrict__ a,
                                                      int64_t a_stride, const T *__restrict__ w, const T *__restrict__ gate,
                                                      int64_t gate_stride, int M, int N, int K, const Heads &at) {
  constexpr int VEC = 16 / sizeof(T);
  const int head = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = (blockIdx.x * GR_WARPS + warp) * GR_COLS;
  const int m0 = blockIdx.z * GR_ROWS;
  const int rows = min(GR_ROWS, M - m0);
  if (n0 >= N) return;
  const T *wh = w + (static_cast<int64_t>(head) * N + n0) * K;
  float acc[GR_ROWS][GR_COLS] = {};
  // lanes take pieces of VEC consecutive k; K is a multiple of VEC (checked by the launcher).  The weights do not
  // depend on the kernel before this one: a lane's first pieces of them are asked for before the wait for it.
  auto load_weights = [&](float (&wv)[GR_COLS][VEC], int k) {
#pragma unroll
    for (int c = 0; c < GR_COLS; ++c) {
      if (n0 + c < N && k < K) {
        const uint4 raw = *reinterpret_cast<const uint4 *>(wh + static_cast<int64_t>(c) * K + k);
        const T *e = reinterpret_cast<const T *>(&raw);
#pragma unroll
        for (int v = 0; v < VEC; ++v) wv[c][v] = le::to_f32(e[v]);
      } else {
#pragma unroll
        for (int v = 0; v < VEC; ++v) wv[c][v] = 0.0f;
      }
    }
  };
  float wv[GR_COLS][VEC];
  load_weights(wv, lane * VEC);
  le::wait_for_predecessor();
  for (int k = lane * VEC; k < K; k += 32 * VEC) {
    if (k != lane * VEC) load_weights(wv, k);
#pragma unroll
    for (int r = 0; r < GR_ROWS; ++r) {
      if (r < rows) {
        const uint4 raw = *reinterpret_cast<const uint4 *>(a + (m0 + r) * a_stride + head * at.a_head + k);
        const T *e = reinterpret_cast<const T *>(&raw);
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          const float x = le::to_f32(e[v]);
#pragma unroll
          for (int c = 0; c < GR_COLS; ++c) acc[r][c] = fmaf(x, wv[c][v], acc[r][c]);
        }
      }
    }
  }
  // The 32 sums over the warp, each in the order of a butterfly over offsets 16, 8, 4, 2, 1; at each offset a lane keeps
  // the half of them that its bit names and hands the other half over, so that lane l ends with sum l (31 exchanges
  // instead of 160).
  static_assert(GR_ROWS * GR_COLS == 32, "a sum per lane");
  float v[32];
#pragma unroll
  for (int i = 0; i < 32; ++i) v[i] = acc[i / GR_COLS][i % GR_COLS];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool upper = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float keep = upper ? v[i + o] : v[i], give = upper ? v[i] : v[i + o];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  const int r = lane / GR_COLS, n = n0 + lane % GR_COLS;
  if (r < rows && n < N) {
    float g = 1.0f;
    if (gate) {
      const int64_t i = (m0 + r) * gate_stride + (at.gate_entries ? static_cast<int64_t>(head) * N + n : head);
      g = 1.0f / (1.0f + expf(-le::to_f32(gate[i])));
    }
    out[(m0 + r) * out_stride + head * at.out_head + n] = le::from_f32<T>(v[0] * g);
  }
}

}  // namespace le_heads
