// Writes of a step's keys and values into the paged cache for mixers whose
// keys carry no position encoding.
//
// kv_store: keys and values are column ranges of the fused projection's rows;
// the token at position p of request b goes to page block_table[b][p / page]
// at offset p % page of pools laid out [pages, kv_heads, page, head_dim].
//
// latent_norm_store: one latent vector per token (a column range of the
// projection's rows, `rank` wide) is divided by its root mean square, times a
// weight, in 32 bits, rounded once, and stored as the single "head" of a pool
// [pages, 1, page, padded_rank]; columns from `rank` on are written as zeros.
// That pool serves as keys and as values of an attention over the latents.
//
// latent_prepare (few rows, a decode step): the latent's norm and store, the
// turns of rotated parts of keys and queries where there are any, and the
// per-head products that carry each head's query into the latent space, in one
// launch: all read the projection's rows and none reads another's
// result.  Blocks whose blockIdx.y is below `heads` do the products, those at
// blockIdx.y == heads walk the tokens' latents, those behind them the queries'
// turns.
#include "gemm_heads_rows.cuh"
#include "latent_token.cuh"

namespace {

template <typename T>
__global__ void kv_store_kernel(const T *__restrict__ src, int64_t src_stride, int k_col, int v_col,
                                T *__restrict__ k_cache, T *__restrict__ v_cache,
                                const int32_t *__restrict__ positions, const int32_t *__restrict__ request_of_token,
                                const int32_t *__restrict__ block_table, int max_blocks, int num_kv_heads, int head_dim,
                                int page_size, int num_pages, int *__restrict__ status) {
  le::let_successor_start();
  le::wait_for_predecessor();
  const int t = blockIdx.x;
  const int pos = positions[t];
  const int b = request_of_token[t];
  const int page = pos >= 0 ? block_table[static_cast<int64_t>(b) * max_blocks + pos / page_size] : -1;
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) atomicOr(status, LE_STATUS_BAD_PAGE);
    return;
  }
  const T *row = src + static_cast<int64_t>(t) * src_stride;
  const int width = num_kv_heads * head_dim;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const int kvh = i / head_dim, d = i - kvh * head_dim;
    const int64_t at = ((static_cast<int64_t>(page) * num_kv_heads + kvh) * page_size + pos % page_size) * head_dim + d;
    k_cache[at] = row[k_col + i];
    v_cache[at] = row[v_col + i];
  }
}

template <typename T>
__global__ void latent_norm_store_kernel(const le_latent::Args<T> a) {
  __shared__ float scratch[33];
  le::let_successor_start();
  le::wait_for_predecessor();
  le_latent::store_latent(a, blockIdx.x, nullptr, scratch);
}

template <typename T>
__global__ void __launch_bounds__(le_heads::GR_WARPS * 32)
latent_prepare_kernel(const le_latent::Args<T> a, int num_tokens, int head_dim, const T *__restrict__ w_into) {
  __shared__ float scratch[33];
  __shared__ float2 turn[le_latent::MAX_PAIRS];
  le::let_successor_start();
  const int part = static_cast<int>(blockIdx.y) - a.heads;
  if (part < 0) {
    // (with a rotated part the product ends at the latent's own columns; without one w_into has rows for the padding too)
    const int N = a.rot > 0 ? a.rank : a.padded;
    le_heads::gemm_heads_rows_block<T>(a.q_out, a.q_stride, a.src, a.src_stride, w_into, static_cast<const T *>(nullptr), 0,
                                       num_tokens, N, head_dim, le_heads::Heads{head_dim + a.rot, a.padded, 0});
    return;
  }
  const bool waits = a.rot == 0;
  if (waits) le::wait_for_predecessor();
  if (part == 0 && a.cache == nullptr) return;
  bool waited = waits;
  // a token to a block, or, of the queries' turns, to as many blocks as there are for it
  const int blocks = gridDim.x * gridDim.z, mine = blockIdx.z * gridDim.x + blockIdx.x;
  const int per = part == 0 ? 1 : max(1, blocks / num_tokens);
  if (mine >= blocks / per * per) return;
  for (int t = mine / per; t < num_tokens; t += blocks / per) {
    if (a.rot > 0) {
      __syncthreads();             // (the last token's turns are done with)
      le_latent::make_turns(turn, a, t);
      if (!waited) le::wait_for_predecessor();
      waited = true;
      __syncthreads();
    }
    if (part == 0) le_latent::store_latent(a, t, turn, scratch);
    else le_latent::turn_queries(a, t, turn, mine % per, per);
  }
}

}  // namespace

// src: rows of stride src_stride; keys start at column k_col, values at v_col, num_kv_heads * head_dim wide each.
LE_API int le_kv_store(const void *src, int64_t src_stride, int k_col, int v_col, void *k_cache, void *v_cache, int dtype,
                       const int32_t *positions, const int32_t *request_of_token, const int32_t *block_table,
                       int max_blocks, int num_tokens, int num_kv_heads, int head_dim, int page_size, int num_pages,
                       int *status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const int width = num_kv_heads * head_dim;
  const int threads = width >= 512 ? 256 : 128;
  LE_DISPATCH_DTYPE(dtype, T,
                    return le::launch_chained(kv_store_kernel<T>, dim3(num_tokens), dim3(threads), 0, stream,
                                              static_cast<const T *>(src), src_stride, k_col, v_col,
                                              static_cast<T *>(k_cache), static_cast<T *>(v_cache), positions,
                                              request_of_token, block_table, max_blocks, num_kv_heads, head_dim,
                                              page_size, num_pages, status));
}

// For at most 32 rows.  src: the projection's rows (stride src_stride, 16-byte aligned): head h's query at columns
// h * (head_dim + rot) .., head_dim plain entries and rot turned ones; the latent at columns col .. col + rank and its
// rotated part behind it.  q_latent[t, h, :] = w_into[h] @ plain part (w_into: [heads, padded_rank, head_dim], or [heads,
// rank, head_dim] where rot > 0) with the turned part behind the rank columns; the latent is normed and stored as
// le_latent_norm_store (rot 0) or le_latent_rope_store does (cache null: not stored).
LE_API int le_latent_prepare(const void *src, int64_t src_stride, int num_tokens, int heads, int head_dim, const void *w_into,
                             void *q_latent, int64_t q_latent_stride, int col, int rank, int rot, int padded_rank,
                             const float *weight, float eps, const void *rates, int rates_wide, float magnitude, void *cache, int dtype,
                             const int32_t *positions, const int32_t *request_of_token, const int32_t *block_table,
                             int max_blocks, int page_size, int num_pages, int *status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const int vec = dtype == LE_BF16 ? 8 : 4;
  if (num_tokens > 32 || head_dim % vec || rot % vec || src_stride % vec || heads < 1 || heads >= 65530 ||
      ((reinterpret_cast<uintptr_t>(src) | reinterpret_cast<uintptr_t>(w_into)) & 15))
    return le::invalid("le_latent_prepare: at most 32 rows, 16-byte aligned rows and head sizes");
  if (rank < 1 || rot < 0 || rot > 2 * le_latent::MAX_PAIRS || padded_rank < rank + rot)
    return le::invalid("le_latent_prepare: rank %d, %d turned entries, padded %d", rank, rot, padded_rank);
  const dim3 grid((padded_rank + le_heads::GR_WARPS * le_heads::GR_COLS - 1) / (le_heads::GR_WARPS * le_heads::GR_COLS),
                  heads + (rot > 0 ? 2 : 1), (num_tokens + le_heads::GR_ROWS - 1) / le_heads::GR_ROWS);
  LE_DISPATCH_DTYPE(dtype, T, {
    le_latent::Args<T> a{static_cast<const T *>(src), src_stride, col, rank, rot, padded_rank, weight, eps, le::Rates{rates, rates_wide}, magnitude,
                         static_cast<T *>(cache), positions, request_of_token, block_table, max_blocks, page_size, num_pages,
                         status, head_dim, head_dim + rot, heads, static_cast<T *>(q_latent), q_latent_stride, 0};
    a.q_pairs = le_latent::pairs_together(a);
    return le::launch_chained(latent_prepare_kernel<T>, grid, dim3(le_heads::GR_WARPS * 32), 0, stream, a, num_tokens, head_dim,
                              static_cast<const T *>(w_into));
  });
}

// src: rows of stride src_stride with the latent at columns col .. col + rank; cache: [pages, 1, page, padded_rank].
LE_API int le_latent_norm_store(const void *src, int64_t src_stride, int col, int rank, int padded_rank,
                                const float *weight, float eps, void *cache, int dtype, const int32_t *positions,
                                const int32_t *request_of_token, const int32_t *block_table, int max_blocks,
                                int num_tokens, int page_size, int num_pages, int *status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (rank < 1 || padded_rank < rank) return le::invalid("le_latent_norm_store: rank %d, padded rank %d", rank, padded_rank);
  const int threads = rank >= 512 ? 256 : 128;
  LE_DISPATCH_DTYPE(dtype, T, {
    const le_latent::Args<T> a{static_cast<const T *>(src), src_stride, col, rank, 0, padded_rank, weight, eps, le::Rates{nullptr, 0}, 1.0f,
                               static_cast<T *>(cache), positions, request_of_token, block_table, max_blocks, page_size,
                               num_pages, status, 0, 0, 0, nullptr, 0, 0};
    return le::launch_chained(latent_norm_store_kernel<T>, dim3(num_tokens), dim3(threads), 0, stream, a);
  });
}
