// Queries, keys and values of a fused projection's rows on their way to the
// attention: bias, a short causal convolution over time on every channel,
// rotary positions on neighbouring pairs of queries and keys, a weightless norm
// per head after the turn, and the paged cache write, in one kernel.
//
// A row holds q [heads, head_dim] | k [kv_heads, head_dim] | v [kv_heads,
// head_dim] (kv_heads 0: queries only, of a layer that reads another layer's
// keys and values).  Per channel, with u = row + bias the projected value:
//
//   y(t) = sum_{j < taps} w[j] * u(t - (taps - 1 - j)),        u before the request's start is zero
//
// then, in every head of q and k, the pair (2i, 2i + 1) below `rot` turns by
// position * rates[i] (cosine and sine times `magnitude`), and the head is divided by sqrt(sum of squares /
// norm_dim + eps) (`unit`).  Queries go to `q_out`, keys and values (these
// neither turned nor normed) to the pages of the token's position.
//
// The taps - 1 projected values before a step are per-request state [taps - 1,
// channels], oldest first, 32-bit, and are brought up to date here.  A lane owns
// its channels: it walks consecutive tokens of one request with the last taps -
// 1 inputs in registers, and only the block that holds a request's first token
// of the step reads that request's state and writes the new one (from the
// step's rows, which this kernel only reads), so no lane reads what another
// writes.  Every step of the sum, the turn and the norm is 32-bit in an order
// that does not depend on how a request is cut; each output is rounded once.
#include "turn.cuh"

namespace {

constexpr int CT_TILE = 16;        // tokens of a tile in the step's lists
constexpr int CT_THREADS = 128;
constexpr int CT_WALK = 4;         // tokens that a lane of the form over 16-byte pieces works on at a time
constexpr int CT_MAX_TAPS = CT_TILE + 1;
constexpr int CT_MAX_PAIRS = 8;    // pairs a lane of the general form holds: heads of up to 512 entries

template <typename T>
struct ConvTurnArgs {
  const T *src;
  int64_t src_stride;
  const float *bias, *taps_w;      // [channels] or null, [taps, channels]
  float *state;                    // [state_rows, taps - 1, channels]
  const int32_t *state_slots, *cu_q, *tile_request, *tile_q0, *positions, *block_table;
  const double *rates;
  T *q_out;
  int64_t q_stride;
  T *k_cache, *v_cache;
  int *status;
  int state_rows, max_blocks, taps, heads, kv_heads, head_dim, rot, unit, norm_dim, page_size, num_pages, write_kv, walk;
  float magnitude, eps;
};

// This block's request and its stretch of tokens: q0 its first (an index among the request's tokens of the step), n of them.
struct Stretch {
  int b, first, q_len, q0, n;
};
template <typename T>
__device__ __forceinline__ Stretch stretch_of(const ConvTurnArgs<T> &a) {
  Stretch s;
  if (a.tile_request != nullptr) {
    const int parts = CT_TILE / a.walk;
    const int tile = blockIdx.x / parts;
    s.b = a.tile_request[tile];
    s.q0 = a.tile_q0[tile] + (blockIdx.x % parts) * a.walk;
    s.first = a.cu_q[s.b], s.q_len = a.cu_q[s.b + 1] - s.first;
  } else {
    s.b = blockIdx.x, s.q0 = 0, s.first = s.b, s.q_len = 1;
  }
  s.n = min(a.walk, s.q_len - s.q0);
  return s;
}
template <typename T>
__device__ __forceinline__ void make_turns(float2 *turn, const ConvTurnArgs<T> &a, const Stretch &s) {
  const int half = a.rot >> 1;
  for (int i = threadIdx.x; i < s.n * half; i += CT_THREADS) {
    const int t = i / half, j = i - t * half;
    turn[i] = le::turn_of(a.positions[s.first + s.q0 + t], a.rates[j], a.magnitude);
  }
}
// Where the stretch's tokens are stored: places[t] is the token's row of its page's first head, in rows of head_dim
// entries from the pool's start (-1: nowhere).  A head further on is page_size rows further.
template <typename T>
__device__ __forceinline__ void find_places(int64_t *places, const ConvTurnArgs<T> &a, const Stretch &s) {
  for (int t = threadIdx.x; t < s.n; t += CT_THREADS) {
    const int pos = a.positions[s.first + s.q0 + t];
    const int page = pos >= 0 ? a.block_table[static_cast<int64_t>(s.b) * a.max_blocks + pos / a.page_size] : -1;
    const bool bad = page < 0 || page >= a.num_pages;
    if (bad) atomicOr(a.status, LE_STATUS_BAD_PAGE);
    places[t] = bad ? -1 : static_cast<int64_t>(page) * a.kv_heads * a.page_size + pos % a.page_size;
  }
}
// The start of head `h` (a key head or, behind those, a value head) at such a place; null: nowhere.
template <typename T>
__device__ __forceinline__ T *page_place(const ConvTurnArgs<T> &a, int64_t place, int h) {
  if (place < 0) return nullptr;
  const bool is_value = h >= a.heads + a.kv_heads;
  const int kvh = h - a.heads - (is_value ? a.kv_heads : 0);
  return (is_value ? a.v_cache : a.k_cache) + (place + static_cast<int64_t>(kvh) * a.page_size) * a.head_dim;
}

template <int N>
__device__ __forceinline__ void load_floats(float (&d)[N], const float *p) {
#pragma unroll
  for (int i = 0; i < N; i += 4) {
    const float4 v = *reinterpret_cast<const float4 *>(p + i);
    d[i] = v.x, d[i + 1] = v.y, d[i + 2] = v.z, d[i + 3] = v.w;
  }
}
template <int N>
__device__ __forceinline__ void store_floats(float *p, const float (&s)[N]) {
#pragma unroll
  for (int i = 0; i < N; i += 4) *reinterpret_cast<float4 *>(p + i) = make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]);
}

// 16 bytes of a row as floats, and back.
template <int N>
__device__ __forceinline__ void open_piece(float (&d)[N], const uint4 &r) {
  const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if constexpr (N == 8) d[2 * i] = __uint_as_float(w[i] << 16), d[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    else d[i] = __uint_as_float(w[i]);
  }
}
template <int N>
__device__ __forceinline__ uint4 close_piece(const float (&v)[N], float f) {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if constexpr (N == 8) {
      const __nv_bfloat162 two = __floats2bfloat162_rn(v[2 * i] * f, v[2 * i + 1] * f);
      w[i] = *reinterpret_cast<const uint32_t *>(&two);
    } else {
      w[i] = __float_as_uint(v[i] * f);
    }
  }
  return make_uint4(w[0], w[1], w[2], w[3]);
}

// 16 bytes of a head per lane (heads of at most 32 such pieces, 2 to 4 taps, everything on 16-byte addresses): a head
// belongs to `lph` neighbouring lanes (a power of two), so a block takes CT_THREADS / lph heads of its stretch.  A lane
// keeps its weights and the last TAPS - 1 inputs in registers, walks its tokens CT_WALK at a time, and asks for the next
// ones' rows before it works on these.
template <typename T, int TAPS>
__global__ void __launch_bounds__(CT_THREADS)
conv_turn_pieces_kernel(const ConvTurnArgs<T> a, int lph) {
  constexpr int N = le::Piece16<T>::COUNT, KEEP = TAPS - 1;
  extern __shared__ float2 turn[];       // [tokens of the stretch][rot / 2]: cosine, sine
  __shared__ int64_t places[CT_TILE];
  le::let_successor_start();
  const Stretch s = stretch_of(a);
  if (s.n <= 0) return;
  const int channels = (a.heads + 2 * a.kv_heads) * a.head_dim;
  const int h = blockIdx.y * (CT_THREADS / lph) + threadIdx.x / lph;
  const int at = (threadIdx.x % lph) * N;                   // first entry of the head that this lane holds
  const bool live = h < a.heads + 2 * a.kv_heads && at < a.head_dim;
  const bool is_query = h < a.heads, is_value = h >= a.heads + a.kv_heads;
  const int turned = is_value || !live ? 0 : a.rot - at;     // this lane's entries below it turn
  const int c = live ? h * a.head_dim + at : 0;
  float w[TAPS][N], bias[N];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) load_floats<N>(w[j], a.taps_w + static_cast<int64_t>(j) * channels + c);
#pragma unroll
  for (int e = 0; e < N; ++e) bias[e] = 0.0f;
  if (a.bias != nullptr) load_floats<N>(bias, a.bias + c);
  make_turns(turn, a, s);
  if (a.write_kv) find_places(places, a, s);
  float *mine = nullptr;
  if (s.q0 == 0 && live) {
    const int slot = a.state_slots[s.b];
    if (slot >= 0 && slot < a.state_rows) mine = a.state + (static_cast<int64_t>(slot) * KEEP) * channels + c;
  }
  le::wait_for_predecessor();
  const T *rows = a.src + static_cast<int64_t>(s.first) * a.src_stride + c;
  auto fetch = [&](uint4 (&raw)[CT_WALK], int i0) {
#pragma unroll
    for (int i = 0; i < CT_WALK; ++i)
      if (i0 + i < s.n) raw[i] = *reinterpret_cast<const uint4 *>(rows + (s.q0 + i0 + i) * a.src_stride);
  };
  uint4 next[CT_WALK];
  fetch(next, 0);
  float past[KEEP][N];
  auto fetch_past = [&](int q) {         // the KEEP inputs before token q of the step
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      open_piece<N>(past[j], *reinterpret_cast<const uint4 *>(rows + (q - KEEP + j) * a.src_stride));
#pragma unroll
      for (int e = 0; e < N; ++e) past[j][e] += bias[e];
    }
  };
  if (s.q0 > 0) {                        // (a stretch that is not the first begins at a multiple of CT_WALK >= KEEP)
    fetch_past(s.q0);
  } else {
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
#pragma unroll
      for (int e = 0; e < N; ++e) past[j][e] = 0.0f;
      if (mine != nullptr) load_floats<N>(past[j], mine + static_cast<int64_t>(j) * channels);
    }
  }
  __syncthreads();                       // turns and places are there
  const float2 *my_turn = turn + (at >> 1);
  const int half = a.rot >> 1;
  const float count = 1.0f / static_cast<float>(a.norm_dim);
  T *q_row = a.q_out + static_cast<int64_t>(s.first + s.q0) * a.q_stride + c;
#pragma unroll 1
  for (int i0 = 0; i0 < s.n; i0 += CT_WALK) {
    uint4 raw[CT_WALK];
#pragma unroll
    for (int i = 0; i < CT_WALK; ++i) raw[i] = next[i];
    fetch(next, i0 + CT_WALK);
#pragma unroll
    for (int i = 0; i < CT_WALK; ++i) {
      if (i0 + i < s.n) {                // (the same for the whole block)
        float u[N], y[N];
        open_piece<N>(u, raw[i]);
#pragma unroll
        for (int e = 0; e < N; ++e) {
          u[e] += bias[e];
          float acc = w[0][e] * past[0][e];
#pragma unroll
          for (int j = 1; j < KEEP; ++j) acc = fmaf(w[j][e], past[j][e], acc);
          y[e] = fmaf(w[KEEP][e], u[e], acc);
        }
#pragma unroll
        for (int e = 0; e < N; ++e) {
#pragma unroll
          for (int j = 0; j + 1 < KEEP; ++j) past[j][e] = past[j + 1][e];
          past[KEEP - 1][e] = u[e];
        }
        if (turned > 0) {
#pragma unroll
          for (int e = 0; e < N; e += 2)
            if (e < turned) le::turn_pair(y[e], y[e + 1], my_turn[(e >> 1)]);
        }
        my_turn += half;
        float inv = 1.0f;
        if (a.unit) {
          float ss = 0.0f;
          if (live) {
#pragma unroll
            for (int e = 0; e < N; ++e) ss = fmaf(y[e], y[e], ss);
          }
          for (int o = 1; o < lph; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
          if (!is_value) inv = rsqrtf(fmaf(ss, count, a.eps));
        }
        T *dst = nullptr;
        if (live && is_query) dst = q_row;
        else if (live && a.write_kv) {
          dst = page_place(a, places[i0 + i], h);
          if (dst != nullptr) dst += at;
        }
        q_row += a.q_stride;
        if (dst != nullptr) *reinterpret_cast<uint4 *>(dst) = close_piece<N>(y, inv);
      }
    }
  }
  if (mine == nullptr) return;
  if (s.q_len > s.n) fetch_past(s.q_len);       // the request goes on beyond this stretch: its last inputs are further down the rows
#pragma unroll
  for (int j = 0; j < KEEP; ++j) store_floats<N>(mine + static_cast<int64_t>(j) * channels, past[j]);
}

// Every other size: a warp per head walks the tokens of a tile; a lane holds every 32nd pair of it and fetches the inputs
// of each tap again.
template <typename T>
__global__ void __launch_bounds__(CT_THREADS)
conv_turn_kernel(const ConvTurnArgs<T> a) {
  extern __shared__ float2 turn[];
  __shared__ int64_t places[CT_TILE];
  le::let_successor_start();
  const Stretch s = stretch_of(a);
  if (s.n <= 0) return;
  const int channels = (a.heads + 2 * a.kv_heads) * a.head_dim, keep = a.taps - 1, half = a.rot >> 1;
  make_turns(turn, a, s);
  if (a.write_kv) find_places(places, a, s);
  le::wait_for_predecessor();
  __syncthreads();
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.y * (CT_THREADS / 32) + (threadIdx.x >> 5);
  if (h >= a.heads + 2 * a.kv_heads) return;              // (whole warps)
  const bool is_query = h < a.heads, is_value = h >= a.heads + a.kv_heads;
  const int pairs = a.head_dim >> 1;
  float *mine = nullptr;
  if (s.q0 == 0 && keep > 0) {
    const int slot = a.state_slots[s.b];
    if (slot >= 0 && slot < a.state_rows) mine = a.state + (static_cast<int64_t>(slot) * keep) * channels;
  }
  // the projected value of channel c at token q of the step (before it: the state, or nothing)
  auto input = [&](int q, int c) {
    if (q >= 0) return le::to_f32(a.src[(s.first + q) * a.src_stride + c]) + (a.bias != nullptr ? a.bias[c] : 0.0f);
    return mine != nullptr ? mine[static_cast<int64_t>(keep + q) * channels + c] : 0.0f;
  };
  for (int i = 0; i < s.n; ++i) {
    float u[CT_MAX_PAIRS], v[CT_MAX_PAIRS];
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < CT_MAX_PAIRS; ++k) {
      const int p = lane + 32 * k;
      if (p < pairs) {
        const int c = h * a.head_dim + 2 * p;
        float acc_u = 0.0f, acc_v = 0.0f;
        for (int j = 0; j <= keep; ++j) {
          const float *wj = a.taps_w + static_cast<int64_t>(j) * channels + c;
          acc_u = fmaf(wj[0], input(s.q0 + i - (keep - j), c), acc_u);
          acc_v = fmaf(wj[1], input(s.q0 + i - (keep - j), c + 1), acc_v);
        }
        if (!is_value && 2 * p + 1 < a.rot) le::turn_pair(acc_u, acc_v, turn[i * half + p]);
        u[k] = acc_u, v[k] = acc_v;
        ss = fmaf(acc_u, acc_u, fmaf(acc_v, acc_v, ss));
      }
    }
    float inv = 1.0f;
    if (a.unit && !is_value) inv = rsqrtf(le::warp_sum(ss) / static_cast<float>(a.norm_dim) + a.eps);
    T *dst = nullptr;
    const int t = s.first + s.q0 + i;
    if (is_query) dst = a.q_out + static_cast<int64_t>(t) * a.q_stride + static_cast<int64_t>(h) * a.head_dim;
    else if (a.write_kv) dst = page_place(a, places[i], h);
    if (dst == nullptr) continue;
#pragma unroll
    for (int k = 0; k < CT_MAX_PAIRS; ++k) {
      const int p = lane + 32 * k;
      if (p < pairs) dst[2 * p] = le::from_f32<T>(u[k] * inv), dst[2 * p + 1] = le::from_f32<T>(v[k] * inv);
    }
  }
  if (mine == nullptr) return;
  // the new state, oldest first (row j comes from row j + q_len of the old one where the step is short: not yet written)
  for (int j = 0; j < keep; ++j) {
    for (int p = lane; p < pairs; p += 32) {
      const int c = h * a.head_dim + 2 * p;
      const float x0 = input(s.q_len - keep + j, c), x1 = input(s.q_len - keep + j, c + 1);
      mine[static_cast<int64_t>(j) * channels + c] = x0, mine[static_cast<int64_t>(j) * channels + c + 1] = x1;
    }
  }
}

}  // namespace

// src: [tokens] rows of src_stride elements, q | k | v heads of head_dim entries (even, at most 512); bias: float32
// [channels] or null; taps_w: float32 [taps, channels], the last row the current token's; state: float32 [state_rows,
// taps - 1, channels] (null when taps is 1); the tile lists name CT_TILE tokens each, or are null when every request
// brings one token (num_tiles requests); rates: float64 [rot / 2]; q_out: rows of q_stride elements, heads * head_dim
// written; k_cache / v_cache: [num_pages, kv_heads, page_size, head_dim].
LE_API int le_conv_turn_store(const void *src, int64_t src_stride, int dtype, const float *bias, const float *taps_w, int taps,
                              float *state, int state_rows, const int32_t *state_slots, const int32_t *cu_q,
                              const int32_t *tile_request, const int32_t *tile_q0, int num_tiles, int tile,
                              const double *rates, int rot, float magnitude, int unit, float eps, int norm_dim, void *q_out,
                              int64_t q_stride, void *k_cache, void *v_cache, const int32_t *positions,
                              const int32_t *block_table, int max_blocks, int heads, int kv_heads, int head_dim, int page_size,
                              int num_pages, int write_kv, int *status, cudaStream_t stream) {
  if (num_tiles <= 0) return 0;
  if (tile != CT_TILE) return le::invalid("le_conv_turn_store: the tiles must list %d tokens each, not %d", CT_TILE, tile);
  if (taps < 1 || taps > CT_MAX_TAPS) return le::invalid("le_conv_turn_store: taps must be 1..%d, got %d", CT_MAX_TAPS, taps);
  if (taps > 1 && state == nullptr) return le::invalid("le_conv_turn_store: %d taps need state", taps);
  if (heads < 1 || kv_heads < 0 || head_dim < 2 || head_dim % 2 || head_dim > 64 * CT_MAX_PAIRS)
    return le::invalid("le_conv_turn_store: heads of %d entries (even, at most %d)", head_dim, 64 * CT_MAX_PAIRS);
  if (rot < 0 || rot % 2 || rot > head_dim) return le::invalid("le_conv_turn_store: %d turned entries in heads of %d", rot, head_dim);
  if (unit && norm_dim < 1) return le::invalid("le_conv_turn_store: the norm needs the entries it runs over");
  if ((tile_request == nullptr) != (tile_q0 == nullptr)) return le::invalid("le_conv_turn_store: both tile lists or neither");
  const int all = heads + 2 * kv_heads, channels = all * head_dim;
  if (src_stride < channels || src == q_out) return le::invalid("le_conv_turn_store: rows of %lld elements hold no %d channels, or are the output", (long long)src_stride, channels);
  const auto on16 = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const int piece = dtype == LE_BF16 ? 8 : 4;
  const bool pieces = taps >= 2 && taps <= 4 && head_dim % piece == 0 && head_dim <= 32 * piece && src_stride % piece == 0 &&
                      q_stride % piece == 0 && on16(src) && on16(q_out) && on16(bias) && on16(taps_w) && on16(state) &&
                      on16(k_cache) && on16(v_cache);
  int lph = 1;
  while (lph * piece < head_dim) lph <<= 1;
  const int per_block = pieces ? CT_THREADS / lph : CT_THREADS / 32;
  // a whole tile to a block where that leaves every multiprocessor a block, else shorter stretches and more blocks
  const bool many = static_cast<int64_t>(num_tiles) * ((all + per_block - 1) / per_block) >= 148;
  const int walk = pieces && !many ? CT_WALK : CT_TILE;
  const dim3 grid(num_tiles * (tile_request == nullptr ? 1 : CT_TILE / walk), (all + per_block - 1) / per_block);
  if (grid.y > 65535) return le::invalid("le_conv_turn_store: %d heads are too many for one launch", all);
  const size_t smem = sizeof(float2) * (tile_request == nullptr ? 1 : walk) * (rot > 0 ? rot / 2 : 1);
  LE_DISPATCH_DTYPE(dtype, T, {
    ConvTurnArgs<T> a;
    a.src = static_cast<const T *>(src), a.src_stride = src_stride, a.bias = bias, a.taps_w = taps_w, a.state = state;
    a.state_slots = state_slots, a.cu_q = cu_q, a.tile_request = tile_request, a.tile_q0 = tile_q0, a.positions = positions;
    a.block_table = block_table, a.rates = rates, a.q_out = static_cast<T *>(q_out), a.q_stride = q_stride;
    a.k_cache = static_cast<T *>(k_cache), a.v_cache = static_cast<T *>(v_cache), a.status = status, a.state_rows = state_rows;
    a.max_blocks = max_blocks, a.taps = taps, a.heads = heads, a.kv_heads = kv_heads, a.head_dim = head_dim, a.rot = rot;
    a.unit = unit, a.norm_dim = norm_dim, a.page_size = page_size, a.num_pages = num_pages, a.write_kv = write_kv;
    a.walk = walk, a.magnitude = magnitude, a.eps = eps;
    if (!pieces) return le::launch_chained(conv_turn_kernel<T>, grid, dim3(CT_THREADS), smem, stream, a);
    auto kernel = taps == 2 ? conv_turn_pieces_kernel<T, 2> : taps == 3 ? conv_turn_pieces_kernel<T, 3> : conv_turn_pieces_kernel<T, 4>;
    return le::launch_chained(kernel, grid, dim3(CT_THREADS), smem, stream, a, lph);
  });
}
