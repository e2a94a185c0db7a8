// A sub-layer's output that enters the residual stream through a norm of its
// own, and the norm of the stream behind it, as one kernel ("norm before and
// after each sub-layer"):
//
//   y' = y + b_in                                              (b_in: the product's bias, optional)
//   x += (y' - mean_y) / sqrt(var_y + eps_y) * w_y + b_y       (the stream, 32-bit, written back)
//   out = (x - mean_x) / sqrt(var_x + eps) * w + b
//
// with var the mean of the squared deviations.  Either norm may leave the
// centring out (mean = 0: a root mean square norm) and either bias may be
// absent.  A factor on what enters the stream is a factor on w_y and b_y.
// Without y the stream is normed as it is.  With a row list only those rows
// are normed, into consecutive rows of `out`, and the stream in memory stays as
// it is.
//
// Everything is 32-bit; `out` is rounded once.  A row is read once: a thread
// keeps its pieces of four values in registers, takes their mean and sum of
// squared deviations exactly in two passes over the registers, and the
// threads' (count, mean, sum of squares) meet pairwise (the parallel update of
// Chan, Golub and LeVeque), so that one meeting of the block makes a norm and a
// mean far from zero costs no digits.
#include "addend.cuh"

namespace {

using le::Addend;
using le::addend4;
using le::addend_at;
using le::load4;
using le::on16;
using le::store4;

struct Moments {
  float n, mean, m2;
};
// Symmetric in its arguments bit for bit, so that the two lanes of an exchange agree.
__device__ __forceinline__ Moments meet(const Moments &a, const Moments &b) {
  const float n = a.n + b.n;
  if (n == 0.0f) return Moments{0.0f, 0.0f, 0.0f};
  const float inv = __fdividef(1.0f, n);
  const float d = a.mean - b.mean;
  const float share = __fmul_rn(__fmul_rn(a.n, b.n), inv);
  return Moments{n, __fmul_rn(__fadd_rn(__fmul_rn(a.n, a.mean), __fmul_rn(b.n, b.mean)), inv),
                 __fmaf_rn(__fmul_rn(d, d), share, __fadd_rn(a.m2, b.m2))};
}
__device__ __forceinline__ Moments meet_lane(const Moments &m, int o) {
  return meet(m, Moments{__shfl_xor_sync(0xffffffffu, m.n, o), __shfl_xor_sync(0xffffffffu, m.mean, o),
                         __shfl_xor_sync(0xffffffffu, m.m2, o)});
}
// The same where both sides have the same count.
__device__ __forceinline__ Moments meet_even(const Moments &m, int o) {
  const float other = __shfl_xor_sync(0xffffffffu, m.mean, o), d = m.mean - other;
  const float m2 = __fadd_rn(m.m2, __shfl_xor_sync(0xffffffffu, m.m2, o));
  return Moments{2.0f * m.n, 0.5f * __fadd_rn(m.mean, other), __fmaf_rn(__fmul_rn(d, d), 0.5f * m.n, m2)};
}
// The block's moments, the same in every thread.  `place`: one Moments per warp, used by one call only.  EVEN: every thread
// brings the same count.
template <bool EVEN = false>
__device__ __forceinline__ Moments block_moments(Moments m, Moments *place) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    if constexpr (EVEN) m = meet_even(m, o);
    else m = meet_lane(m, o);
  }
  if (warps == 1) return m;
  if (lane == 0) place[warp] = m;
  __syncthreads();
  if (EVEN && (warps & (warps - 1)) == 0) {        // (every lane reads a warp's and all end with the same)
    m = place[lane & (warps - 1)];
    for (int o = 1; o < warps; o <<= 1) m = meet_even(m, o);
    return m;
  }
  m = lane < warps ? place[lane] : Moments{0.0f, 0.0f, 0.0f};
  for (int o = 1; o < 16; o <<= 1) m = meet_lane(m, o);          // (at most 16 warps, in lanes 0 .. 15)
  m.n = __shfl_sync(0xffffffffu, m.n, 0), m.mean = __shfl_sync(0xffffffffu, m.mean, 0), m.m2 = __shfl_sync(0xffffffffu, m.m2, 0);
  return m;
}

struct NormArgs {
  const float *w, *b;      // b may be null
  float eps;
  int centered;
};

__device__ __forceinline__ void add4(float4 &a, const float4 &b) { a.x += b.x, a.y += b.y, a.z += b.z, a.w += b.w; }

template <int V, bool EVEN = false>
__device__ __forceinline__ Moments thread_moments(const float4 (&v)[V], int n4, bool centered) {
  if constexpr (EVEN) {
    float sum = 0.0f, m2 = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) sum += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    const float mean = centered ? sum * (0.25f / V) : 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float a = v[i].x - mean, b = v[i].y - mean, c = v[i].z - mean, d = v[i].w - mean;
      m2 = fmaf(a, a, fmaf(b, b, fmaf(c, c, fmaf(d, d, m2))));
    }
    return Moments{4.0f * V, mean, m2};
  }
  int count = 0;
  float sum = 0.0f;
#pragma unroll
  for (int i = 0; i < V; ++i) {
    if (static_cast<int>(threadIdx.x + i * blockDim.x) < n4) count += 4, sum += (v[i].x + v[i].y) + (v[i].z + v[i].w);
  }
  const float mean = centered && count ? sum * (V == 1 ? 0.25f : 1.0f / static_cast<float>(count)) : 0.0f;
  float m2 = 0.0f;
#pragma unroll
  for (int i = 0; i < V; ++i) {
    if (static_cast<int>(threadIdx.x + i * blockDim.x) < n4) {
      const float a = v[i].x - mean, b = v[i].y - mean, c = v[i].z - mean, d = v[i].w - mean;
      m2 = fmaf(a, a, fmaf(b, b, fmaf(c, c, fmaf(d, d, m2))));
    }
  }
  return Moments{static_cast<float>(count), mean, m2};
}

__device__ __forceinline__ float4 normed4(const float4 &v, float mean, float inv, const float4 &w, const float4 &b) {
  return make_float4(fmaf((v.x - mean) * inv, w.x, b.x), fmaf((v.y - mean) * inv, w.y, b.y),
                     fmaf((v.z - mean) * inv, w.z, b.z), fmaf((v.w - mean) * inv, w.w, b.w));
}

// Rows whose pieces of four fit V to a thread, everything on 16-byte addresses.  PARTS: the addend's partial sums where
// that number is known when compiling (0: as `y` says), so that all of a thread's loads are in flight together.  AHEAD:
// the weights are asked for before the wait for the kernel before this one (few rows, where that time counts).
template <typename T, int V, int PARTS, bool AHEAD>
__global__ void __launch_bounds__(AHEAD ? 512 : 256)
addend_norm_kernel(T *__restrict__ out, float *__restrict__ resid, Addend y, const float *__restrict__ b_in, NormArgs ny,
                   NormArgs nx, const int32_t *__restrict__ rows, int width) {
  __shared__ Moments places[2][16];
  le::let_successor_start();
  const int n4 = width >> 2;
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  float4 wx[V], bx[V], wy[V], by[V], bi[V];
  auto fetch = [&](float4 (&d)[V], const float *p) {
#pragma unroll
    for (int v = 0; v < V; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      d[v] = p != nullptr && i < n4 ? load4(p + 4 * i) : zero;
    }
  };
  if constexpr (AHEAD) {
    if (y.data != nullptr) fetch(bi, b_in), fetch(wy, ny.w), fetch(by, ny.b);
    fetch(wx, nx.w), fetch(bx, nx.b);
  }
  le::wait_for_predecessor();
  const int64_t r = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
  float *x = resid + r * width;
  float4 xv[V];
  fetch(xv, x);
  if (y.data != nullptr) {
    float4 yv[V];
    if constexpr (PARTS > 1) {
      float4 part[V][PARTS];
      const float *p = static_cast<const float *>(y.data) + r * width;
#pragma unroll
      for (int s = 0; s < PARTS; ++s) {
#pragma unroll
        for (int v = 0; v < V; ++v) {
          const int i = threadIdx.x + v * blockDim.x;
          part[v][s] = i < n4 ? load4(p + s * y.part_stride + 4 * i) : zero;
        }
      }
#pragma unroll
      for (int v = 0; v < V; ++v) {
        yv[v] = part[v][0];
#pragma unroll
        for (int s = 1; s < PARTS; ++s) add4(yv[v], part[v][s]);
      }
    } else {
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const int i = threadIdx.x + v * blockDim.x;
        yv[v] = i < n4 ? addend4(y, r * width + 4 * i) : zero;
      }
    }
    if constexpr (!AHEAD) fetch(bi, b_in);
#pragma unroll
    for (int v = 0; v < V; ++v) add4(yv[v], bi[v]);
    const Moments m = block_moments(thread_moments<V>(yv, n4, ny.centered), places[0]);
    const float inv = rsqrtf(m.m2 / static_cast<float>(width) + ny.eps);
    if constexpr (!AHEAD) fetch(wy, ny.w), fetch(by, ny.b);
#pragma unroll
    for (int v = 0; v < V; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      add4(xv[v], normed4(yv[v], m.mean, inv, wy[v], by[v]));
      if (rows == nullptr && i < n4) store4(x + 4 * i, xv[v]);
    }
  }
  const Moments m = block_moments(thread_moments<V>(xv, n4, nx.centered), places[1]);
  const float inv = rsqrtf(m.m2 / static_cast<float>(width) + nx.eps);
  if constexpr (!AHEAD) fetch(wx, nx.w), fetch(bx, nx.b);
  T *o = out + static_cast<int64_t>(blockIdx.x) * width;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int i = threadIdx.x + v * blockDim.x;
    if (i < n4) store4(o + 4 * i, normed4(xv[v], m.mean, inv, wx[v], bx[v]));
  }
}

// BYTES (8 or 16) from global to shared memory without passing through registers; done when asked_for() says so.
template <int BYTES>
__device__ __forceinline__ void ask_for(void *dst, const void *src) {
  const uint32_t at = static_cast<uint32_t>(__cvta_generic_to_shared(dst));
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2;\n" ::"r"(at), "l"(src), "n"(BYTES) : "memory");
}
__device__ __forceinline__ void close_group() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int LEFT>
__device__ __forceinline__ void asked_for() { asm volatile("cp.async.wait_group %0;\n" ::"n"(LEFT) : "memory"); }

// Many rows with an addend of one tensor, two pieces of four to a thread: as many blocks as the device holds at once walk
// the rows, with the weights in registers and the next rows on their way into a ring in shared memory (a thread reads back
// only what it asked for itself, so the ring needs no barrier).
constexpr int RING = 4;
template <typename T, typename TD, bool EVEN>
__global__ void __launch_bounds__(512)
addend_norm_rows_kernel(T *__restrict__ out, float *__restrict__ resid, const TD *__restrict__ y, const float *__restrict__ b_in,
                        NormArgs ny, NormArgs nx, int n, int width) {
  constexpr int V = 2, Y_BYTES = 4 * sizeof(TD);
  __shared__ Moments places[2][16];
  extern __shared__ __align__(16) unsigned char ring[];        // [RING][V][threads] pieces of x, then of y
  float4 *x_ring = reinterpret_cast<float4 *>(ring);
  unsigned char *y_ring = ring + sizeof(float4) * RING * V * blockDim.x;
  le::let_successor_start();
  const int n4 = width >> 2;
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  float4 wx[V], bx[V], wy[V], by[V], bi[V];
  auto fetch = [&](float4 (&d)[V], const float *p) {
#pragma unroll
    for (int v = 0; v < V; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      d[v] = p != nullptr && i < n4 ? load4(p + 4 * i) : zero;
    }
  };
  fetch(bi, b_in), fetch(wy, ny.w), fetch(by, ny.b), fetch(wx, nx.w), fetch(bx, nx.b);
  le::wait_for_predecessor();
  auto ask = [&](int r, int stage) {          // (a group per row, also an empty one)
    if (r < n) {
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const int i = threadIdx.x + v * blockDim.x;
        if (EVEN || i < n4) {
          const int at = (stage * V + v) * blockDim.x + threadIdx.x;
          ask_for<16>(x_ring + at, resid + static_cast<int64_t>(r) * width + 4 * i);
          ask_for<Y_BYTES>(y_ring + Y_BYTES * at, y + static_cast<int64_t>(r) * width + 4 * i);
        }
      }
    }
    close_group();
  };
#pragma unroll
  for (int s = 0; s < RING - 1; ++s) ask(blockIdx.x + s * gridDim.x, s);
  int stage = 0;
  const float share = 1.0f / static_cast<float>(width);
  for (int r = blockIdx.x; r < n; r += gridDim.x) {
    ask(r + (RING - 1) * static_cast<int>(gridDim.x), (stage + RING - 1) % RING);
    asked_for<RING - 1>();
    float4 xv[V], yv[V];
#pragma unroll
    for (int v = 0; v < V; ++v) {
      const bool mine = EVEN || static_cast<int>(threadIdx.x + v * blockDim.x) < n4;
      const int at = (stage * V + v) * blockDim.x + threadIdx.x;
      xv[v] = mine ? x_ring[at] : zero;
      yv[v] = mine ? load4(reinterpret_cast<const TD *>(y_ring + Y_BYTES * at)) : zero;
      add4(yv[v], bi[v]);
    }
    stage = (stage + 1) % RING;
    // (a place is written again only behind the other one's barrier, when every thread has read it)
    Moments m = block_moments<EVEN>(thread_moments<V, EVEN>(yv, n4, ny.centered), places[0]);
    float inv = rsqrtf(fmaf(m.m2, share, ny.eps));
#pragma unroll
    for (int v = 0; v < V; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      add4(xv[v], normed4(yv[v], m.mean, inv, wy[v], by[v]));
      if (EVEN || i < n4) store4(resid + static_cast<int64_t>(r) * width + 4 * i, xv[v]);
    }
    m = block_moments<EVEN>(thread_moments<V, EVEN>(xv, n4, nx.centered), places[1]);
    inv = rsqrtf(fmaf(m.m2, share, nx.eps));
    T *o = out + static_cast<int64_t>(r) * width;
#pragma unroll
    for (int v = 0; v < V; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      if (EVEN || i < n4) store4(o + 4 * i, normed4(xv[v], m.mean, inv, wx[v], bx[v]));
    }
  }
}

// Any width: the row in shared memory, two passes over it per norm.
template <typename T>
__global__ void __launch_bounds__(256)
addend_norm_any_kernel(T *__restrict__ out, float *__restrict__ resid, Addend y, const float *__restrict__ b_in, NormArgs ny,
                       NormArgs nx, const int32_t *__restrict__ rows, int width) {
  extern __shared__ float row[];
  __shared__ float scratch[33];
  le::let_successor_start();
  le::wait_for_predecessor();
  const int64_t r = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
  float *x = resid + r * width;
  auto moments = [&](bool centered, float &mean, float &inv, float eps) {
    mean = 0.0f;
    if (centered) {
      float sum = 0.0f;
      for (int i = threadIdx.x; i < width; i += blockDim.x) sum += row[i];
      mean = le::block_sum(sum, scratch) / static_cast<float>(width);
    }
    float sq = 0.0f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) sq = fmaf(row[i] - mean, row[i] - mean, sq);
    inv = rsqrtf(le::block_sum(sq, scratch) / static_cast<float>(width) + eps);
  };
  float mean, inv;
  if (y.data != nullptr) {
    for (int i = threadIdx.x; i < width; i += blockDim.x)        // (a thread reads back only what it wrote)
      row[i] = addend_at(y, r * width + i) + (b_in != nullptr ? b_in[i] : 0.0f);
    moments(ny.centered, mean, inv, ny.eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
      row[i] = x[i] + fmaf((row[i] - mean) * inv, ny.w[i], ny.b != nullptr ? ny.b[i] : 0.0f);
      if (rows == nullptr) x[i] = row[i];
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] = x[i];
  }
  moments(nx.centered, mean, inv, nx.eps);
  T *o = out + static_cast<int64_t>(blockIdx.x) * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x)
    o[i] = le::from_f32<T>(fmaf((row[i] - mean) * inv, nx.w[i], nx.b != nullptr ? nx.b[i] : 0.0f));
}

template <typename T, typename TD, bool EVEN>
int launch_rows(T *out, float *resid, const void *y, const float *b_in, const NormArgs &ny, const NormArgs &nx, int n, int width,
                int threads, cudaStream_t stream) {
  auto kernel = addend_norm_rows_kernel<T, TD, EVEN>;
  const size_t smem = static_cast<size_t>(RING) * 2 * threads * (sizeof(float4) + 4 * sizeof(TD));
  static int resident[17] = {};                  // blocks the device holds at once, by warps to a block
  int &blocks = resident[threads / 32];
  if (blocks == 0) {
    int device = 0, sms = 0, per_sm = 0;
    cudaGetDevice(&device);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
    cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, RING * 2 * 512 * (sizeof(float4) + 4 * sizeof(TD)));
    cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, kernel, threads, smem);
    blocks = sms * per_sm > 0 ? sms * per_sm : 1;
  }
  const int rounds = (n + blocks - 1) / blocks;
  return le::launch_chained(kernel, dim3((n + rounds - 1) / rounds), dim3(threads), smem, stream, out, resid,
                            static_cast<const TD *>(y), b_in, ny, nx, n, width);
}

template <typename T, int V, bool AHEAD>
int launch_parts(T *out, float *resid, const Addend &y, const float *b_in, const NormArgs &ny, const NormArgs &nx,
                 const int32_t *rows, int n, int width, int threads, cudaStream_t stream) {
#define LE_GO(PARTS)                                                                                                    \
  return le::launch_chained(addend_norm_kernel<T, V, PARTS, AHEAD>, dim3(n), dim3(threads), 0, stream, out, resid, y, b_in, \
                            ny, nx, rows, width)
  if constexpr (AHEAD) {
    if (y.data != nullptr && y.dtype == LE_F32) {
      if (y.parts == 2) LE_GO(2);
      if (y.parts == 3) LE_GO(3);
      if (y.parts == 4) LE_GO(4);
    }
  }
  LE_GO(0);
#undef LE_GO
}

}  // namespace

// resid [rows, width] float32; y: an addend (y_parts partial sums y_stride elements apart) or null; b_in [width] or null;
// w_y, b_y [width]: the addend's norm (b_y null: none; both null only without an addend), y_centered: whether its mean
// is taken off; w, b, centered: the stream's norm; out [n, width] in the type `out_dtype`; all vectors float32.
LE_API int le_addend_norm(void *out, int out_dtype, float *resid, const void *y, int y_dtype, int y_parts, int64_t y_stride,
                          const float *b_in, const float *w_y, const float *b_y, float eps_y, int y_centered, const float *w,
                          const float *b, float eps, int centered, const int32_t *rows, int n, int width, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width < 1 || width > 32 * 1024) return le::invalid("le_addend_norm: rows of %d values (at most 32768)", width);
  if (out == nullptr || w == nullptr || (y != nullptr && w_y == nullptr)) return le::invalid("le_addend_norm: a norm needs its weight");
  const Addend add{y, y_dtype, y_parts < 1 ? 1 : y_parts, y_stride};
  const NormArgs ny{w_y, b_y, eps_y, y_centered}, nx{w, b, eps, centered};
  if (width % 4 == 0 && width <= 8192 && y_stride % 4 == 0 && on16(out) && on16(resid) && on16(y) && on16(b_in) && on16(w_y) &&
      on16(b_y) && on16(w) && on16(b)) {
    const int n4 = width / 4;
    // few rows: a row is one round of loads of up to 512 threads; many: smaller blocks, several to a multiprocessor
    const bool few = n <= 148 && width <= 4096;
    int threads = (n4 + 31) / 32 * 32;
    const int most = few ? 512 : 256;
    threads = threads > most ? most : threads;
    const int per = (n4 + threads - 1) / threads;
    if (!few && y != nullptr && rows == nullptr && add.parts == 1 && n4 > 128 && n4 <= 1024) {
      const int half = ((n4 + 1) / 2 + 31) / 32 * 32;
      const bool even = n4 == 2 * half;
#define LE_ROWS(T, TD)                                                                                                       \
  return even ? launch_rows<T, TD, true>(static_cast<T *>(out), resid, y, b_in, ny, nx, n, width, half, stream)               \
              : launch_rows<T, TD, false>(static_cast<T *>(out), resid, y, b_in, ny, nx, n, width, half, stream)
      if (out_dtype == LE_BF16 && y_dtype == LE_BF16) LE_ROWS(__nv_bfloat16, __nv_bfloat16);
      if (out_dtype == LE_F32 && y_dtype == LE_F32) LE_ROWS(float, float);
#undef LE_ROWS
    }
#define LE_V(V, AHEAD)                                                                                                       \
  LE_DISPATCH_DTYPE(out_dtype, T,                                                                                            \
                    return launch_parts<T, V, AHEAD>(static_cast<T *>(out), resid, add, b_in, ny, nx, rows, n, width, threads, stream))
    if (per <= 1) { if (few) LE_V(1, true); LE_V(1, false); }
    if (per <= 2) { if (few) LE_V(2, true); LE_V(2, false); }
    if (per <= 4) LE_V(4, false);
    LE_V(8, false);
#undef LE_V
  }
  const size_t smem = sizeof(float) * width;
  LE_DISPATCH_DTYPE(out_dtype, T,
                    if (smem > 40 * 1024) cudaFuncSetAttribute(addend_norm_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
                    return le::launch_chained(addend_norm_any_kernel<T>, dim3(n), dim3(256), smem, stream, static_cast<T *>(out),
                                              resid, add, b_in, ny, nx, rows, width));
}
