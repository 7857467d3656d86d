// The cached side of a latent attention: a token's compressed key/value vector.
//
// A layer with a down-projection of its own turns each token's projection (rank numbers) into
// c = x / sqrt(mean(x^2) + eps) * gain and keeps only c, in a paged cache with one "head" of
// size rank and no separate values.  Keys and values of every head are linear maps of c, so the
// attention itself runs on c: the queries are first carried through the key map
// (q'_h = Wuk_h^T q_h, so that q_h . k_h = q'_h . c), the attention is then a multi-query one whose
// keys and values are both c, and its result is carried through the value map afterwards.  This
// file holds the norm-and-store step; the two per-head maps are batched products (gemm_simt.cu)
// and the attention is the paged multi-query kernels that the other mixers use.
#include "common.cuh"

namespace {

constexpr int WARPS = 4;

// One warp per token: sum of squares, reciprocal root and scaling in float32; the result is
// rounded to the cache's element type once and written at the token's place in the pages.
template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
latent_norm_store_kernel(const T* __restrict__ x, long long x_stride, const float* __restrict__ gain, float eps,
                         const int* __restrict__ slot_map, T* __restrict__ pages, int n_tokens, int rank, int row_width) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * WARPS + warp;
  if (t >= n_tokens) return;
  const T* row = x + (size_t)t * x_stride;
  float ss = 0.f;
  for (int c = lane; c < rank; c += 32) {
    const float v = to_f32(row[c]);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  const float r = 1.f / sqrtf(ss / (float)rank + eps);
  T* dst = pages + (size_t)slot_map[t] * row_width;
  for (int c = lane; c < rank; c += 32) dst[c] = from_f32<T>(to_f32(row[c]) * r * gain[c]);
  for (int c = rank + lane; c < row_width; c += 32) dst[c] = from_f32<T>(0.f);      // a row wider than the rank ends in zeros
}


// The same for a latent attention with a query latent and a rotated key part: one warp per token takes the token's
// projection x = [query latent: q_rank | key/value latent: rank | rotated key part: rot] (float32) and writes
//   cq = rms(x_q) * q_gain                                        to cq_out (the element kind of the step), and
//   [rotated key part | rms(x_c) * gain | zeros]                   to the token's cache row:
// the pairs (2i, 2i + 1), i < pairs, of the key part turn by position * freqs[i] (one float32 product, sincosf); what lies
// beyond them passes; amp multiplies cos and sin.  The rotated part comes first in the row so that the kernels that turn the leading channels of a
// head serve the queries too.
template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
latent_rope_norm_store_kernel(const float* __restrict__ x, long long x_stride, const float* __restrict__ q_gain, int q_rank,
                              T* __restrict__ cq_out, long long cq_stride, const float* __restrict__ gain, int rank, int rot,
                              const float* __restrict__ freqs, int pairs, const int* __restrict__ positions, float eps,
                              const int* __restrict__ slot_map, T* __restrict__ pages, int n_tokens, int row_width, float amp) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * WARPS + warp;
  if (t >= n_tokens) return;
  const float* row = x + (size_t)t * x_stride;
  if (q_rank > 0) {
    float ss = 0.f;
    for (int c = lane; c < q_rank; c += 32) ss = fmaf(row[c], row[c], ss);
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)q_rank + eps);
    for (int c = lane; c < q_rank; c += 32) cq_out[(size_t)t * cq_stride + c] = from_f32<T>(row[c] * r * q_gain[c]);
  }
  if (pages == nullptr) return;
  const float* lat = row + q_rank;
  const float* kr = lat + rank;
  float ss = 0.f;
  for (int c = lane; c < rank; c += 32) ss = fmaf(lat[c], lat[c], ss);
  const float r = 1.f / sqrtf(warp_sum(ss) / (float)rank + eps);
  T* dst = pages + (size_t)slot_map[t] * row_width;
  const float pos = (float)positions[t];
  for (int i = lane; i < rot / 2; i += 32) {
    float u = kr[2 * i], v = kr[2 * i + 1];
    if (i < pairs) {
      float sn, cs;
      sincosf(pos * freqs[i], &sn, &cs);
      sn *= amp; cs *= amp;
      const float u2 = u * cs - v * sn, v2 = v * cs + u * sn;
      u = u2; v = v2;
    }
    dst[2 * i] = from_f32<T>(u);
    dst[2 * i + 1] = from_f32<T>(v);
  }
  for (int c = lane; c < rank; c += 32) dst[rot + c] = from_f32<T>(lat[c] * r * gain[c]);
  for (int c = rot + rank + lane; c < row_width; c += 32) dst[c] = from_f32<T>(0.f);
}

// Queries and latents from one product: a token's row of x (float32, or the unsummed split-K partial results) is
//   [ heads x (rot turned | dim plain) | latent: rank | rotated key part: rot ]
// The leading pairs (2i, 2i + 1), i < pairs, of every head and of the key part turn by position * freqs[i] (one float32
// product, sincosf; amp multiplies cos and sin); the queries go to q_out in the element kind, and the token's cache row
// [turned key part | rms(latent) * gain | zeros] to its place in the pages.  pages null: a layer that reads another's latents,
// its row holds the queries alone.  Grid (tokens, parts): part 0 writes the cache row, all parts share the query channels.
constexpr int QL_THREADS = 256;

template <typename T, bool VEC>
__global__ void __launch_bounds__(QL_THREADS)
latent_q_rope_store_kernel(MaybePartial<float> x, long long x_stride, T* __restrict__ q_out, long long q_stride, int heads, int dim,
                           const float* __restrict__ gain, int rank, int rot, const float* __restrict__ freqs, int pairs, float amp,
                           const int* __restrict__ positions, float eps, const int* __restrict__ slot_map, T* __restrict__ pages,
                           int row_width) {
  __shared__ float cs_s[512], sn_s[512], red[32];
  extern __shared__ float lat_s[];            // [rank], part 0 with pages
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x;
  const size_t row = (size_t)t * x_stride;
  const float pos = (float)positions[t];
  for (int i = tid; i < pairs; i += QL_THREADS) {
    float sn, cs;
    sincosf(pos * freqs[i], &sn, &cs);
    sn_s[i] = sn * amp; cs_s[i] = cs * amp;
  }
  __syncthreads();
  if (VEC) {                                  // eight channels a thread, 16-byte accesses (rot and dim multiples of 8)
    const int per8 = (rot + dim) / 8;
    for (int idx = blockIdx.y * QL_THREADS + tid; idx < heads * per8; idx += gridDim.y * QL_THREADS) {
      const int i = idx % per8 * 4;           // the piece's first pair within its head
      float u[8];
      x.at8(row + (size_t)idx * 8, u);
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (i + k < pairs) {
          const float a = u[2 * k], b = u[2 * k + 1];
          u[2 * k] = a * cs_s[i + k] - b * sn_s[i + k];
          u[2 * k + 1] = b * cs_s[i + k] + a * sn_s[i + k];
        }
      Vec8<T>::store(q_out + (size_t)t * q_stride + (size_t)idx * 8, u);
    }
  }
  // two neighbouring channels a thread: every head is an even number of channels before its plain part, which may end odd
  const int per = rot + dim, half = (per + 1) / 2;
  for (int idx = blockIdx.y * QL_THREADS + tid; !VEC && idx < heads * half; idx += gridDim.y * QL_THREADS) {
    const int h = idx / half, i = idx - h * half, c = 2 * i;
    const size_t at = row + (size_t)h * per + c;
    float u = x.at(at), v = c + 1 < per ? x.at(at + 1) : 0.f;
    if (i < pairs) {
      const float u2 = u * cs_s[i] - v * sn_s[i], v2 = v * cs_s[i] + u * sn_s[i];
      u = u2; v = v2;
    }
    T* dst = q_out + (size_t)t * q_stride + (size_t)h * per + c;
    dst[0] = from_f32<T>(u);
    if (c + 1 < per) dst[1] = from_f32<T>(v);
  }
  if (pages == nullptr || blockIdx.y != 0) return;
  const size_t lat = row + (size_t)heads * per, kr = lat + rank;
  float ss = 0.f;
  for (int c = tid; c < rank; c += QL_THREADS) {
    const float v = x.at(lat + c);
    lat_s[c] = v;                             // read back by the thread that wrote it
    ss = fmaf(v, v, ss);
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)rank + eps);
  T* dst = pages + (size_t)slot_map[t] * row_width;
  for (int i = tid; i < rot / 2; i += QL_THREADS) {
    float u = x.at(kr + 2 * i), v = x.at(kr + 2 * i + 1);
    if (i < pairs) {
      const float u2 = u * cs_s[i] - v * sn_s[i], v2 = v * cs_s[i] + u * sn_s[i];
      u = u2; v = v2;
    }
    dst[2 * i] = from_f32<T>(u);
    dst[2 * i + 1] = from_f32<T>(v);
  }
  for (int c = tid; c < rank; c += QL_THREADS) dst[rot + c] = from_f32<T>(lat_s[c] * r * gain[c]);
  for (int c = rot + rank + tid; c < row_width; c += QL_THREADS) dst[c] = from_f32<T>(0.f);
}

}  // namespace

// x float32 [n_tokens, x_stride] or its partial results [splits][n_tokens][x_stride]; see latent_q_rope_store_kernel.  q_out
// [n_tokens, q_stride] with heads * (rot + dim) columns; rot even, pairs <= rot / 2, at most 512.
LLMK_API int llmk_latent_q_rope_store(const float* x, const float* partials, int splits, long long split_stride, long long x_stride,
                                      void* q_out, long long q_stride, int heads, int dim, const float* gain, int rank, int rot,
                                      const float* freqs, int pairs, float amp, const int* positions, float eps, const int* slot_map,
                                      void* pages, int n_tokens, int row_width, int dtype, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  LLMK_REQUIRE((x != nullptr) != (partials != nullptr), "latent_q_rope_store: give x or partials");
  LLMK_REQUIRE(heads > 0 && dim > 0 && rot >= 0 && rot % 2 == 0 && pairs >= 0 && 2 * pairs <= rot && pairs <= 512,
               "latent_q_rope_store: bad sizes: %d heads of %d + %d channels, %d pairs", heads, rot, dim, pairs);
  LLMK_REQUIRE(pages == nullptr || (rank > 0 && rank <= 8192 && row_width >= rot + rank), "latent_q_rope_store: bad rank %d or row width %d", rank, row_width);
  // few tokens: a token's channels are spread over several CTAs
  const int items = heads * ((rot + dim + 7) / 8);
  const int parts = n_tokens >= 256 ? 1 : max(1, min(16, (items + QL_THREADS - 1) / QL_THREADS));
  return dispatch_dtype(dtype, [&](auto* tag) {
    using T = LLMK_ELEM(tag);
    MaybePartial<float> src{x, partials, splits, split_stride};
    const bool vec = rot % 8 == 0 && dim % 8 == 0 && src.vector_ok() && x_stride % 8 == 0 && q_stride % 8 == 0 && (uintptr_t)q_out % 16 == 0;
    launch_kernel(vec ? latent_q_rope_store_kernel<T, true> : latent_q_rope_store_kernel<T, false>, dim3(n_tokens, parts), dim3(QL_THREADS),
                  pages ? (size_t)rank * sizeof(float) : 0, stream, src, x_stride, (T*)q_out, q_stride, heads, dim, gain, rank, rot, freqs,
                  pairs, amp, positions, eps, slot_map, (T*)pages, row_width);
    LLMK_LAUNCH_CHECK("latent_q_rope_store");
  });
}

// x [n_tokens, x_stride]: the first `rank` columns of a row are the token's projection.
// pages [pages, 1, page_size, row_width] with row_width >= rank (a cache whose rows are padded to a width
// that the attention kernels take; the padding is written as zeros); slot_map[t] = page * page_size + offset.
LLMK_API int llmk_latent_norm_store(const void* x, long long x_stride, const float* gain, float eps,
                                    const int* slot_map, void* pages, int n_tokens, int rank, int row_width, int dtype,
                                    cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  LLMK_REQUIRE(rank > 0 && x_stride >= rank && row_width >= rank, "latent_norm_store: bad rank %d, width %d or stride %lld", rank, row_width, x_stride);
  return dispatch_dtype(dtype, [&](auto* tag) {
    using T = LLMK_ELEM(tag);
    launch_kernel(latent_norm_store_kernel<T>, dim3((n_tokens + WARPS - 1) / WARPS), dim3(WARPS * 32), 0, stream,
                  (const T*)x, x_stride, gain, eps, slot_map, (T*)pages, n_tokens, rank, row_width);
    LLMK_LAUNCH_CHECK("latent_norm_store");
  });
}

// x float32 [n_tokens, x_stride]: [q_rank | rank | rot] per row (q_rank 0: no query latent; pages null: no cache row, a
// layer that reads another's).  rot is even; pairs <= rot / 2.  pages [pages, 1, page_size, row_width], row_width >= rot + rank.
LLMK_API int llmk_latent_rope_norm_store(const float* x, long long x_stride, const float* q_gain, int q_rank, void* cq_out,
                                         long long cq_stride, const float* gain, int rank, int rot, const float* freqs, int pairs,
                                         const int* positions, float eps, const int* slot_map, void* pages, int n_tokens,
                                         int row_width, int dtype, cudaStream_t stream, float amp) {
  if (n_tokens == 0) return 0;
  LLMK_REQUIRE(rank > 0 && rot >= 0 && rot % 2 == 0 && 2 * pairs <= rot && q_rank >= 0,
               "latent_rope_norm_store: bad rank %d, rotated size %d, pairs %d or query rank %d", rank, rot, pairs, q_rank);
  LLMK_REQUIRE(pages == nullptr || row_width >= rot + rank, "latent_rope_norm_store: a row of %d is too narrow", row_width);
  return dispatch_dtype(dtype, [&](auto* tag) {
    using T = LLMK_ELEM(tag);
    launch_kernel(latent_rope_norm_store_kernel<T>, dim3((n_tokens + WARPS - 1) / WARPS), dim3(WARPS * 32), 0, stream, x, x_stride,
                  q_gain, q_rank, (T*)cq_out, cq_stride, gain, rank, rot, freqs, pairs, positions, eps, slot_map, (T*)pages,
                  n_tokens, row_width, amp);
    LLMK_LAUNCH_CHECK("latent_rope_norm_store");
  });
}
