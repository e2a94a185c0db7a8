// Linear attention with one fixed decay per head (lightning attention) over the
// step's tokens, request by request, from each request's state row and back
// into it.  Per head, with q, k [dim] and v [vdim] after their activation:
//
//   S <- decay * S + k v^T                 o = S^T q
//
// S is float32 in memory ([state rows, heads, vdim, dim]) and in registers.
//
// scan: token by token, any type and size.  A block takes one request, one
// head and ROWS of the vdim columns of S; a column has LANES threads, each with
// every LANES-th group of four entries in registers.  Tokens pass in tiles
// through shared memory.  The decay comes in
// two floats whose sum is the 64-bit number: its rounding to one float would lean
// the same way at every token, and a memory of a thousand tokens would be off
// by a thousand times that.  This is the kernel of decoded tokens, which is
// bound by reading and writing S.
//
// chunks: the same sums by chunks of 64 tokens on the tensor cores (bfloat16
// q, k, v; heads of up to 128 entries), for requests that bring several
// tokens.  With p(n) = decay^n and i, j the places within a chunk of L tokens:
//
//   o_i = p(i + 1) S^T q_i + sum_{j <= i} p(i - j) (q_i . k_j) v_j
//   S  <- p(L) S + sum_j p(L - 1 - j) k_j v_j^T
//
// q, k and v are exact bfloat16 operands; the 32-bit numbers that meet them in
// a product (S, the weighted scores, the weighted keys) are split into two
// bfloat16 parts, high and low, and both parts are multiplied, so that they
// keep 16 bits of mantissa or more; all sums are 32-bit, and S itself is never
// rounded.  A segment of SEGMENT tokens is a block's work (one head, 64 of the vdim
// columns).  A request of one segment goes from its state row to its state row.
// Requests of several segments take three launches: every segment's own sum
// (S from zero, no outputs) into scratch, the segments' starting states and
// the request's new state row from those sums (element by element), and the
// outputs of every segment from its starting state, all segments side by side.
#include "common.cuh"

namespace {

using bf16 = __nv_bfloat16;

// ---------------------------------------------------------------- scan
constexpr int LS_THREADS = 256;
constexpr int LS_TILE = 16;
constexpr int LS_QUADS = 4;       // groups of four entries a thread holds at most

struct ScanArgs {
  float *out; int64_t out_stride;
  const void *rows; int64_t row_stride; int q_col, k_col, v_col;
  const float *decay;             // [2, heads]: high parts, low parts
  float *state; int num_state_rows;
  const int32_t *state_slots, *cu_q;
  const int32_t *requests;        // the requests this launch takes, or null: all in order
  int heads, dim, vdim, rows_per_block, tile;
};

template <typename T, int LANES>
__global__ void __launch_bounds__(LS_THREADS)
lightning_scan_kernel(ScanArgs p) {
  extern __shared__ __align__(16) float ls_smem[];
  const int D = p.dim, DQ = (D + 3) / 4 * 4, ROWS = p.rows_per_block;
  float *s_q = ls_smem;                          // [tile][DQ]
  float *s_k = s_q + p.tile * DQ;                // [tile][DQ]
  float *s_v = s_k + p.tile * DQ;                // [tile][ROWS]
  float *s_o = s_v + p.tile * ROWS;              // [tile][ROWS]
  le::let_successor_start();
  const int b = p.requests != nullptr ? p.requests[blockIdx.z] : blockIdx.z;
  const int head = blockIdx.y, e0 = blockIdx.x * ROWS;
  const int r = threadIdx.x / LANES, lane = threadIdx.x % LANES;
  const int cols = min(ROWS, p.vdim - e0);
  const int first = p.cu_q[b], q_len = p.cu_q[b + 1] - first;
  const int slot = p.state_slots[b];
  const bool has_state = slot >= 0 && slot < p.num_state_rows;
  const bool active = r < cols && has_state;
  const int threads = blockDim.x;
  const float high = p.decay[head], low = p.decay[p.heads + head];
  float *mine = active ? p.state + ((static_cast<int64_t>(slot) * p.heads + head) * p.vdim + e0 + r) * D : nullptr;
  const bool quads = D % 4 == 0;                 // (rows of the state then start on 16 bytes)
  float S[LS_QUADS][4];
#pragma unroll
  for (int j = 0; j < LS_QUADS; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.0f;
  le::wait_for_predecessor();
  if (active) {
#pragma unroll
    for (int j = 0; j < LS_QUADS; ++j) {
      const int d = 4 * (lane + LANES * j);
      if (d >= D) continue;
      if (quads) {
        const float4 v = *reinterpret_cast<const float4 *>(mine + d);
        S[j][0] = v.x, S[j][1] = v.y, S[j][2] = v.z, S[j][3] = v.w;
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (d + e < D) S[j][e] = mine[d + e];
      }
    }
  }
  const T *rows = static_cast<const T *>(p.rows);

  for (int t0 = 0; t0 < q_len; t0 += p.tile) {
    const int tile = min(p.tile, q_len - t0);
    __syncthreads();                             // the tile before is stored
    for (int i = threadIdx.x; i < tile * DQ; i += threads) {
      const int t = i / DQ, d = i - t * DQ;
      const T *row = rows + static_cast<int64_t>(first + t0 + t) * p.row_stride + static_cast<int64_t>(head) * D + d;
      s_q[i] = d < D ? le::to_f32(row[p.q_col]) : 0.0f;
      s_k[i] = d < D ? le::to_f32(row[p.k_col]) : 0.0f;
    }
    for (int i = threadIdx.x; i < tile * ROWS; i += threads) {
      const int t = i / ROWS, c = i - t * ROWS;
      s_v[i] = c < cols ? le::to_f32(rows[static_cast<int64_t>(first + t0 + t) * p.row_stride + p.v_col +
                                     static_cast<int64_t>(head) * p.vdim + e0 + c]) : 0.0f;
    }
    __syncthreads();
    for (int t = 0; t < tile; ++t) {
      const float v = r < ROWS ? s_v[t * ROWS + r] : 0.0f;
      float acc = 0.0f;
#pragma unroll
      for (int j = 0; j < LS_QUADS; ++j) {
        const int d = 4 * (lane + LANES * j);
        if (d >= D) continue;
        const float4 k = *reinterpret_cast<const float4 *>(s_k + t * DQ + d);
        const float4 q = *reinterpret_cast<const float4 *>(s_q + t * DQ + d);
        S[j][0] = fmaf(high, S[j][0], fmaf(low, S[j][0], k.x * v));
        S[j][1] = fmaf(high, S[j][1], fmaf(low, S[j][1], k.y * v));
        S[j][2] = fmaf(high, S[j][2], fmaf(low, S[j][2], k.z * v));
        S[j][3] = fmaf(high, S[j][3], fmaf(low, S[j][3], k.w * v));
        acc = fmaf(S[j][0], q.x, fmaf(S[j][1], q.y, fmaf(S[j][2], q.z, fmaf(S[j][3], q.w, acc))));
      }
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
      if (lane == 0 && r < ROWS) s_o[t * ROWS + r] = acc;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < tile * ROWS; i += threads) {
      const int t = i / ROWS, c = i - t * ROWS;
      if (c < cols)
        p.out[static_cast<int64_t>(first + t0 + t) * p.out_stride + static_cast<int64_t>(head) * p.vdim + e0 + c] =
            has_state ? s_o[i] : 0.0f;
    }
  }
  if (active) {
#pragma unroll
    for (int j = 0; j < LS_QUADS; ++j) {
      const int d = 4 * (lane + LANES * j);
      if (d >= D) continue;
      if (quads) {
        *reinterpret_cast<float4 *>(mine + d) = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (d + e < D) mine[d + e] = S[j][e];
      }
    }
  }
}

template <typename T, int LANES>
int launch_scan(const ScanArgs &p, int num_requests, cudaStream_t stream) {
  const dim3 grid((p.vdim + p.rows_per_block - 1) / p.rows_per_block, p.heads, num_requests);
  // (whole warps: the lanes of a column meet by shuffles)
  const int threads = (p.rows_per_block * LANES + 31) / 32 * 32;
  const size_t smem = sizeof(float) * p.tile * (2 * ((p.dim + 3) / 4 * 4) + 2 * p.rows_per_block);
  if (smem > 48 * 1024) {
    static size_t raised = 0;                    // per form and process: the most asked for so far
    if (smem > raised) {
      cudaError_t e = cudaFuncSetAttribute(lightning_scan_kernel<T, LANES>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
      if (e != cudaSuccess) return le::invalid("le_lightning_scan: cannot get %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
      raised = smem;
    }
  }
  return le::launch_chained(lightning_scan_kernel<T, LANES>, grid, dim3(threads), smem, stream, p);
}

// ---------------------------------------------------------------- chunks
constexpr int CHUNK = 64;
constexpr int SEGMENT = 256;
constexpr int LC_COLS = 64;       // columns of S a block takes
constexpr int LC_THREADS = 256;
constexpr int LC_LDV = LC_COLS + 8;

__device__ __forceinline__ uint32_t smem_addr(const void *p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const bf16 *p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], const bf16 *p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two floats as two bfloat16 pairs whose sum keeps 16 bits of each.
__device__ __forceinline__ void split_pair(float x, float y, uint32_t &high, uint32_t &low) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  high = *reinterpret_cast<const uint32_t *>(&h);
  low = *reinterpret_cast<const uint32_t *>(&l);
}
__device__ __forceinline__ float low_of(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float high_of(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }

struct ChunkArgs {
  float *out; int64_t out_stride;
  const bf16 *rows; int64_t row_stride; int q_col, k_col, v_col;
  const float *powers;            // [heads, SEGMENT + 1]: decay^n
  float *state; int num_state_rows;
  float *scratch;                 // [segments, heads, vdim, dim], or null: every request is one segment
  const int32_t *state_slots, *cu_q, *tile_request, *tile_q0;
  int heads, dim, vdim, vector;   // vector: 16-byte pieces are whole and aligned
};

template <int DP, bool SUMS>
constexpr size_t chunk_smem() {
  return sizeof(bf16) * ((SUMS ? 2 : 3) * CHUNK * (DP + 8) + 2 * CHUNK * LC_LDV + (SUMS ? 0 : 2 * DP * LC_LDV)) +
         sizeof(float) * (CHUNK + 4);
}

// DP: the heads' entries, padded to a multiple of 32 (zeros behind the real ones).  SUMS: only the segment's own sum
// into scratch.  Eight warps: for the outputs warp w has the 16 tokens (w % 4) and 32 of the columns (w / 4); for the
// state it has DP / 16 of the 16 x 8 tiles of S, in order of their rows.
template <int DP, bool SUMS>
__global__ void __launch_bounds__(LC_THREADS, 2)
lightning_chunk_kernel(ChunkArgs p) {
  extern __shared__ __align__(16) unsigned char lc_smem[];
  constexpr int LD = DP + 8;
  constexpr int NT = LC_COLS / 8;                  // 8-column tiles of S
  constexpr int TILES = DP / 16 * NT / 8;          // tiles of S a warp holds
  constexpr int KSTEPS = DP / 16;
  bf16 *s_q = reinterpret_cast<bf16 *>(lc_smem);   // [CHUNK][LD]
  bf16 *s_k = s_q + (SUMS ? 0 : CHUNK * LD);       // [2][CHUNK][LD]
  bf16 *s_v = s_k + 2 * CHUNK * LD;                // [2][CHUNK][LC_LDV]
  bf16 *s_sh = s_v + 2 * CHUNK * LC_LDV;           // [DP][LC_LDV]: S, high parts
  bf16 *s_sl = s_sh + DP * LC_LDV;                 // low parts
  float *s_pow = reinterpret_cast<float *>(SUMS ? s_sh : s_sl + DP * LC_LDV);      // [CHUNK + 1]
  le::let_successor_start();
  const int slices = (p.vdim + LC_COLS - 1) / LC_COLS;
  const int head = blockIdx.x / slices, e0 = (blockIdx.x % slices) * LC_COLS;
  const int seg = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t4 = lane & 3, j8 = lane >> 3, r8 = lane & 7;
  const int D = p.dim, cols = min(LC_COLS, p.vdim - e0);
  for (int i = tid; i <= CHUNK; i += LC_THREADS) s_pow[i] = p.powers[head * (SEGMENT + 1) + i];
  le::wait_for_predecessor();
  const int b = p.tile_request[seg], q0 = p.tile_q0[seg];
  const int tokens = min(SEGMENT, p.cu_q[b + 1] - p.cu_q[b] - q0);
  const int64_t first = p.cu_q[b] + q0;
  const int slot = p.state_slots[b];
  const bool has_state = slot >= 0 && slot < p.num_state_rows;

  // S in accumulator fragments: tile i of this warp is rows 16 m .. + 15, columns 8 n .. + 7
  float acc_s[TILES][4];
  auto tile_row = [&](int i) { return (warp * TILES + i) / NT * 16; };
  auto tile_col = [&](int i) { return (warp * TILES + i) % NT * 8; };
  float *from = nullptr;
  if (!SUMS) {
    if (p.scratch != nullptr) from = p.scratch + (static_cast<int64_t>(seg) * p.heads + head) * p.vdim * D;
    else if (has_state) from = p.state + (static_cast<int64_t>(slot) * p.heads + head) * p.vdim * D;
  }
#pragma unroll
  for (int i = 0; i < TILES; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = tile_row(i) + g + (e >> 1) * 8, c = tile_col(i) + 2 * t4 + (e & 1);
      acc_s[i][e] = from != nullptr && d < D && c < cols ? from[static_cast<int64_t>(e0 + c) * D + d] : 0.0f;
    }

  // A chunk's rows, copied straight into shared memory while the chunk before is worked on: k and v have two buffers,
  // q one (it is free once the fragments are in registers).  Rows beyond the tokens and entries beyond the sizes: zeros.
  auto copy_rows = [&](bf16 *dst, int ld, int pieces, int col, int limit, int c0) {
    for (int id = tid; id < CHUNK * pieces; id += LC_THREADS) {
      const int t = id / pieces, at = (id - t * pieces) * 8;
      const bool live = c0 + t < tokens && at < limit;
      const bf16 *src = live ? p.rows + (first + c0 + t) * p.row_stride + col + at : p.rows;
      bf16 *to = dst + t * ld + at;
      if (p.vector) {
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_addr(to)), "l"(src), "r"(live ? 16 : 0) : "memory");
      } else {
#pragma unroll
        for (int u = 0; u < 8; ++u) to[u] = live && at + u < limit ? src[u] : __float2bfloat16_rn(0.0f);
      }
    }
  };
  auto fetch = [&](int c0) {
    const int buffer = (c0 / CHUNK) & 1;
    if constexpr (!SUMS) copy_rows(s_q, LD, DP / 8, p.q_col + head * D, D, c0);
    copy_rows(s_k + buffer * CHUNK * LD, LD, DP / 8, p.k_col + head * D, D, c0);
    copy_rows(s_v + buffer * CHUNK * LC_LDV, LC_LDV, LC_COLS / 8, p.v_col + head * p.vdim + e0, cols, c0);
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  fetch(0);

  for (int c0 = 0; c0 < tokens; c0 += CHUNK) {
    const int L = min(CHUNK, tokens - c0);
    const bf16 *k_at = s_k + ((c0 / CHUNK) & 1) * CHUNK * LD, *v_at = s_v + ((c0 / CHUNK) & 1) * CHUNK * LC_LDV;
    if constexpr (!SUMS) {
#pragma unroll
      for (int i = 0; i < TILES; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          uint32_t high, low;
          split_pair(acc_s[i][2 * h], acc_s[i][2 * h + 1], high, low);
          const int at = (tile_row(i) + g + 8 * h) * LC_LDV + tile_col(i) + 2 * t4;
          *reinterpret_cast<uint32_t *>(s_sh + at) = high;
          *reinterpret_cast<uint32_t *>(s_sl + at) = low;
        }
    }
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();                             // the chunk and the state before it are there
    // this warp's tokens and columns (the later tokens see more keys: the warps of a scheduler share them out)
    const int r0 = 16 * (warp < 4 ? warp : 7 - warp), n0 = 32 * (warp >> 2);
    const bool outputs = !SUMS && r0 < L && n0 < cols;
    uint32_t qf[KSTEPS][4];
    if constexpr (!SUMS) {
      if (outputs) {
#pragma unroll
        for (int ks = 0; ks < KSTEPS; ++ks) ldsm4(qf[ks], s_q + (r0 + (j8 & 1) * 8 + r8) * LD + ks * 16 + (j8 >> 1) * 8);
      }
      __syncthreads();                           // q is in registers
    }
    if (c0 + CHUNK < tokens) fetch(c0 + CHUNK);

    if constexpr (!SUMS) {
      if (outputs) {
        const int row[2] = {r0 + g, r0 + g + 8};
        // what the state before the chunk gives
        float o[4][4];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.0f;
#pragma unroll
        for (int ks = 0; ks < KSTEPS; ++ks)
#pragma unroll
          for (int np = 0; np < 2; ++np) {
            const int at = (ks * 16 + (j8 & 1) * 8 + r8) * LC_LDV + n0 + np * 16 + (j8 >> 1) * 8;
            uint32_t bh[4], bl[4];
            ldsm4_trans(bh, s_sh + at);
            ldsm4_trans(bl, s_sl + at);
            mma(o[2 * np], qf[ks], bl[0], bl[1]);
            mma(o[2 * np + 1], qf[ks], bl[2], bl[3]);
            mma(o[2 * np], qf[ks], bh[0], bh[1]);
            mma(o[2 * np + 1], qf[ks], bh[2], bh[3]);
          }
        const float from_start[2] = {s_pow[row[0] + 1], s_pow[row[1] + 1]};
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          o[nt][0] *= from_start[0], o[nt][1] *= from_start[0];
          o[nt][2] *= from_start[1], o[nt][3] *= from_start[1];
        }
        // the chunk's own keys, 16 at a time up to this warp's tokens
        for (int kb = 0; kb <= r0; kb += 16) {
          float s[2][4] = {};
#pragma unroll
          for (int ks = 0; ks < KSTEPS; ++ks) {
            uint32_t kf[4];
            ldsm4(kf, k_at + (kb + (j8 >> 1) * 8 + r8) * LD + ks * 16 + (j8 & 1) * 8);
            mma(s[0], qf[ks], kf[0], kf[1]);
            mma(s[1], qf[ks], kf[2], kf[3]);
          }
          uint32_t ph[4], pl[4];
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              const int back = row[h] - (kb + nt * 8 + 2 * t4);    // how far the pair's first key lies back
              const float x = back >= 0 ? s[nt][2 * h] * s_pow[back] : 0.0f;
              const float y = back >= 1 ? s[nt][2 * h + 1] * s_pow[back - 1] : 0.0f;
              split_pair(x, y, ph[nt * 2 + h], pl[nt * 2 + h]);
            }
#pragma unroll
          for (int np = 0; np < 2; ++np) {
            uint32_t vf[4];
            ldsm4_trans(vf, v_at + (kb + (j8 & 1) * 8 + r8) * LC_LDV + n0 + np * 16 + (j8 >> 1) * 8);
            mma(o[2 * np], pl, vf[0], vf[1]);
            mma(o[2 * np + 1], pl, vf[2], vf[3]);
            mma(o[2 * np], ph, vf[0], vf[1]);
            mma(o[2 * np + 1], ph, vf[2], vf[3]);
          }
        }
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          if (row[h] >= L) continue;
          float *dst = p.out + (first + c0 + row[h]) * p.out_stride + static_cast<int64_t>(head) * p.vdim + e0 + n0 + 2 * t4;
#pragma unroll
          for (int nt = 0; nt < 4; ++nt) {
            const int c = n0 + nt * 8 + 2 * t4;
            const float x = has_state ? o[nt][2 * h] : 0.0f, y = has_state ? o[nt][2 * h + 1] : 0.0f;
            if (p.vector && c + 1 < cols) {
              *reinterpret_cast<float2 *>(dst + nt * 8) = make_float2(x, y);
            } else {
              if (c < cols) dst[nt * 8] = x;
              if (c + 1 < cols) dst[nt * 8 + 1] = y;
            }
          }
        }
      }
    }
    // the state behind the chunk (rows of keys beyond its tokens are zero)
    {
      const float keep = s_pow[L];
#pragma unroll
      for (int i = 0; i < TILES; ++i) acc_s[i][0] *= keep, acc_s[i][1] *= keep, acc_s[i][2] *= keep, acc_s[i][3] *= keep;
#pragma unroll
      for (int kb = 0; kb < CHUNK; kb += 16) {
        if (kb >= L) break;
        // this lane's tokens of the 16: kb + 2 t4, + 1, + 8, + 9
        float f[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int t = kb + 2 * t4 + (u & 1) + (u >> 1) * 8;
          f[u] = t < L ? s_pow[L - 1 - t] : 0.0f;
        }
        uint32_t ah[4], al[4];
        int have = -1;
#pragma unroll
        for (int i = 0; i < TILES; i += 2) {
          const bool pair = i + 1 < TILES;
          if (tile_row(i) != have) {
            have = tile_row(i);
            uint32_t kf[4];
            ldsm4_trans(kf, k_at + (kb + (j8 >> 1) * 8 + r8) * LD + have + (j8 & 1) * 8);
#pragma unroll
            for (int u = 0; u < 4; ++u)
              split_pair(low_of(kf[u]) * f[(u >> 1) * 2], high_of(kf[u]) * f[(u >> 1) * 2 + 1], ah[u], al[u]);
          }
          uint32_t vf[4];
          ldsm4_trans(vf, v_at + (kb + (j8 & 1) * 8 + r8) * LC_LDV + tile_col(i) + (j8 >> 1) * 8);
          mma(acc_s[i], al, vf[0], vf[1]);
          if (pair) mma(acc_s[i + 1], al, vf[2], vf[3]);
          mma(acc_s[i], ah, vf[0], vf[1]);
          if (pair) mma(acc_s[i + 1], ah, vf[2], vf[3]);
        }
      }
    }
    __syncthreads();                             // everyone is done with this chunk's keys and values and with S
  }

  float *to = nullptr;
  if (SUMS) to = p.scratch + (static_cast<int64_t>(seg) * p.heads + head) * p.vdim * D;
  else if (p.scratch == nullptr && has_state) to = p.state + (static_cast<int64_t>(slot) * p.heads + head) * p.vdim * D;
  if (to == nullptr) return;
#pragma unroll
  for (int i = 0; i < TILES; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = tile_row(i) + g + (e >> 1) * 8, c = tile_col(i) + 2 * t4 + (e & 1);
      if (d < D && c < cols) to[static_cast<int64_t>(e0 + c) * D + d] = acc_s[i][e];
    }
}

// From every segment's own sum: the state each segment starts from (in place of the sums) and the request's new state
// row.  A request's segments stand in the list in their order, other requests' between them; the blocks of its first one
// do its work, a thread for four entries of S (V = 4; 1 where they are no whole pieces), with the sums of eight segments
// asked for at a time.
constexpr int LC_AHEAD = 8;
template <int V>
__global__ void __launch_bounds__(256)
lightning_starts_kernel(ChunkArgs p, int num_segments) {
  le::let_successor_start();
  const int seg = blockIdx.z, head = blockIdx.y;
  const int n = p.vdim * p.dim;
  const int i = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (p.tile_q0[seg] != 0 || i >= n) return;      // (the step's integers are older than the kernel before this one)
  const int b = p.tile_request[seg];
  const int q_len = p.cu_q[b + 1] - p.cu_q[b];
  const int segments = (q_len + SEGMENT - 1) / SEGMENT;
  const float keep = p.powers[head * (SEGMENT + 1) + SEGMENT];
  const float last = p.powers[head * (SEGMENT + 1) + min(SEGMENT, q_len - (segments - 1) * SEGMENT)];
  const int slot = p.state_slots[b];
  const bool has_state = slot >= 0 && slot < p.num_state_rows;
  float *row = has_state ? p.state + (static_cast<int64_t>(slot) * p.heads + head) * n + i : nullptr;
  float *part = p.scratch + static_cast<int64_t>(head) * n + i;       // of segment s of the list: + s * step
  const int64_t step = static_cast<int64_t>(p.heads) * n;
  auto load = [](float (&v)[V], const float *at) {
    if constexpr (V == 4) {
      const float4 r = *reinterpret_cast<const float4 *>(at);
      v[0] = r.x, v[1] = r.y, v[2] = r.z, v[3] = r.w;
    } else {
      v[0] = *at;
    }
  };
  auto store = [](float *at, const float (&v)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4 *>(at) = make_float4(v[0], v[1], v[2], v[3]);
    else *at = v[0];
  };
  le::wait_for_predecessor();
  float S[V];
#pragma unroll
  for (int v = 0; v < V; ++v) S[v] = 0.0f;
  if (row != nullptr) load(S, row);
  int at = seg;                                   // the request's next segment in the list
  for (int s0 = 0; s0 < segments; s0 += LC_AHEAD) {
    float sum[LC_AHEAD][V];
    int where[LC_AHEAD];
#pragma unroll
    for (int u = 0; u < LC_AHEAD; ++u) {
      while (at < num_segments && p.tile_request[at] != b) ++at;
      where[u] = s0 + u < segments && at < num_segments ? at++ : -1;
      if (where[u] >= 0) load(sum[u], part + where[u] * step);
    }
#pragma unroll
    for (int u = 0; u < LC_AHEAD; ++u) {
      if (where[u] < 0) break;
      store(part + where[u] * step, S);
      const float f = s0 + u + 1 < segments ? keep : last;
#pragma unroll
      for (int v = 0; v < V; ++v) S[v] = fmaf(f, S[v], sum[u][v]);
    }
  }
  if (row != nullptr) store(row, S);
}

template <int DP, bool SUMS>
int launch_chunks(const ChunkArgs &p, int segments, cudaStream_t stream) {
  constexpr size_t smem = chunk_smem<DP, SUMS>();
  auto kernel = lightning_chunk_kernel<DP, SUMS>;
  if (smem > 48 * 1024) {
    static bool raised = false;                  // once per form and process
    if (!raised) {
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
      if (e != cudaSuccess) return le::invalid("le_lightning_chunks: cannot get %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
      raised = true;
    }
  }
  const dim3 grid(p.heads * ((p.vdim + LC_COLS - 1) / LC_COLS), segments);
  return le::launch_chained(kernel, grid, dim3(LC_THREADS), smem, stream, p);
}

template <int DP>
int run_chunks(const ChunkArgs &p, int segments, cudaStream_t stream) {
  if (p.scratch != nullptr) {
    int rc = launch_chunks<DP, true>(p, segments, stream);
    if (rc != 0) return rc;
    const int n = p.vdim * p.dim;
    const bool quads = n % 4 == 0 && (reinterpret_cast<uintptr_t>(p.scratch) | reinterpret_cast<uintptr_t>(p.state)) % 16 == 0;
    const dim3 grid((n / (quads ? 4 : 1) + 255) / 256, p.heads, segments);
    rc = quads ? le::launch_chained(lightning_starts_kernel<4>, grid, dim3(256), 0, stream, p, segments)
               : le::launch_chained(lightning_starts_kernel<1>, grid, dim3(256), 0, stream, p, segments);
    if (rc != 0) return rc;
  }
  return launch_chunks<DP, false>(p, segments, stream);
}

}  // namespace

// out: float32 [T, heads * vdim].  rows (`dtype`): per token q [heads, dim] at q_col, k at k_col, v [heads, vdim] at
// v_col, after their activation.  decay: float32 [2, heads], the decays' high and low parts.
// state: float32 [num_state_rows, heads, vdim, dim].  requests: the indices of the num_requests requests to run, or
// null: requests 0 .. num_requests - 1.  single: every one of them brings one token (it only chooses the launch's shape).
LE_API int le_lightning_scan(float *out, int64_t out_stride, const void *rows, int64_t row_stride, int q_col, int k_col, int v_col,
                             int dtype, const float *decay, float *state, int num_state_rows,
                             const int32_t *state_slots, const int32_t *cu_q, const int32_t *requests, int num_requests,
                             int heads, int dim, int vdim, int single, cudaStream_t stream) {
  if (num_requests <= 0) return 0;
  if (heads < 1 || dim < 1 || vdim < 1 || heads > 65535 || num_requests > 65535)
    return le::invalid("le_lightning_scan: %d heads of %d x %d for %d requests", heads, dim, vdim, num_requests);
  if (dim > 4 * LS_QUADS * 32) return le::invalid("le_lightning_scan: heads of at most %d entries, got %d", 4 * LS_QUADS * 32, dim);
  int lanes = 1;
  while (4 * LS_QUADS * lanes < dim) lanes *= 2;
  ScanArgs p;
  p.out = out, p.out_stride = out_stride, p.rows = rows, p.row_stride = row_stride, p.q_col = q_col, p.k_col = k_col, p.v_col = v_col;
  p.decay = decay, p.state = state, p.num_state_rows = num_state_rows, p.state_slots = state_slots, p.cu_q = cu_q;
  p.requests = requests, p.heads = heads, p.dim = dim, p.vdim = vdim;
  p.tile = single ? 1 : LS_TILE;
  const int most = LS_THREADS / lanes;
  p.rows_per_block = vdim < most ? vdim : most;
#define LE_SCAN(T)                                                             \
  do {                                                                         \
    switch (lanes) {                                                           \
      case 1: return launch_scan<T, 1>(p, num_requests, stream);               \
      case 2: return launch_scan<T, 2>(p, num_requests, stream);               \
      case 4: return launch_scan<T, 4>(p, num_requests, stream);               \
      case 8: return launch_scan<T, 8>(p, num_requests, stream);               \
      case 16: return launch_scan<T, 16>(p, num_requests, stream);             \
      default: return launch_scan<T, 32>(p, num_requests, stream);             \
    }                                                                          \
  } while (0)
  if (dtype == LE_F32) LE_SCAN(float);
  if (dtype == LE_BF16) LE_SCAN(bf16);
#undef LE_SCAN
  return le::invalid("le_lightning_scan: unknown dtype code %d", dtype);
}

LE_API int le_lightning_segment() { return SEGMENT; }

// The same over chunks, for bfloat16 rows and heads of up to 128 entries.
// tile_request / tile_q0 list num_segments segments of le_lightning_segment() tokens: their requests and their first
// tokens within them, a request's segments in their order (other requests' may stand between them).  powers: float32 [heads, le_lightning_segment() + 1],
// decay^n.  scratch: float32 [num_segments, heads, vdim, dim] where a request has several
// segments, else null.
LE_API int le_lightning_chunks(float *out, int64_t out_stride, const void *rows, int64_t row_stride, int q_col, int k_col,
                               int v_col, const float *powers, float *state, int num_state_rows,
                               float *scratch, const int32_t *state_slots, const int32_t *cu_q, const int32_t *tile_request,
                               const int32_t *tile_q0, int num_segments, int heads, int dim, int vdim, cudaStream_t stream) {
  if (num_segments <= 0) return 0;
  if (heads < 1 || heads > 65535 || dim < 1 || dim > 128 || vdim < 1 || num_segments > 65535)
    return le::invalid("le_lightning_chunks: %d heads of %d x %d in %d segments", heads, dim, vdim, num_segments);
  ChunkArgs p;
  p.out = out, p.out_stride = out_stride, p.rows = static_cast<const bf16 *>(rows), p.row_stride = row_stride;
  p.q_col = q_col, p.k_col = k_col, p.v_col = v_col, p.powers = powers, p.state = state;
  p.num_state_rows = num_state_rows, p.scratch = scratch, p.state_slots = state_slots, p.cu_q = cu_q;
  p.tile_request = tile_request, p.tile_q0 = tile_q0, p.heads = heads, p.dim = dim, p.vdim = vdim;
  p.vector = dim % 8 == 0 && vdim % 8 == 0 && q_col % 8 == 0 && k_col % 8 == 0 && v_col % 8 == 0 && row_stride % 8 == 0 &&
             reinterpret_cast<uintptr_t>(rows) % 16 == 0 && out_stride % 2 == 0 && reinterpret_cast<uintptr_t>(out) % 8 == 0;
  if (dim <= 32) return run_chunks<32>(p, num_segments, stream);
  if (dim <= 64) return run_chunks<64>(p, num_segments, stream);
  if (dim <= 96) return run_chunks<96>(p, num_segments, stream);
  return run_chunks<128>(p, num_segments, stream);
}
