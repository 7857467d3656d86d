// Linear attention with one fixed decay per head:
//
//   S_t = d_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t          S [dim, vdim] per head, float32, in the request's state slot
//
// scan.cu walks it token by token for any sizes (its "const" form).  This file holds the two forms that real sizes run on.
//
// Single tokens (a decode step): the state is read and written once and everything else is small.  A CTA owns 64 columns of
// one head's state; its 128 threads are 16 float4 columns x 8 row lanes; up to 16 rows of a thread are in flight at once.
// q, k and v are read as they left the projection, a tensor or its unsummed split-K partial results, and pass silu here.
//
// Prompt portions (bfloat16): chunks of 64 tokens.  With n tokens in the chunk and S_0 the state that enters it,
//     o_i = d^(i+1) S_0^T q_i + sum_{j <= i} d^(i-j) (q_i . k_j) v_j,       S_n = d^n S_0 + sum_j d^(n-1-j) k_j v_j^T
// so the chunks' own contributions to the state are made side by side (chunk_state), chained from the request's state by one
// multiply-add per chunk and element (chunk_chain, float32), and the outputs are made side by side again (chunk_out).  q, k and
// v are bfloat16 (silu already taken, in the epilogue of the product that made them), so q . k and k v^T have exact factors;
// every float32 operand of a product (the state, the decayed scores, the decayed values) enters it as the sum of three bfloat16
// numbers, which hold its 24 bits, and every sum is float32.  The products are warp-level MMAs (mma.sync): their operands are
// made in registers by the warp that uses them, and a tile is 64 rows.
#include "warp_mma.cuh"

namespace {

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }

// ---- single tokens -----------------------------------------------------------------------------------------
constexpr int DEC_COLS = 64, DEC_TX = DEC_COLS / 4, DEC_ROWS = 8, DEC_THREADS = DEC_TX * DEC_ROWS, DEC_BATCH = 16, DEC_MAX_DIM = 512;

// proj row e: [q: heads * dim | k: heads * dim | v: heads * vdim | ...], pre-activation.  out [e, heads * vdim] float32.
template <typename T>
__global__ void __launch_bounds__(DEC_THREADS)
lightning_decode_kernel(float* __restrict__ out, long long out_stride, MaybePartial<T> proj, long long proj_stride,
                        const float* __restrict__ decay, float* __restrict__ state, long long slot_stride,
                        const int* __restrict__ state_slots, int heads, int dim, int vdim) {
  __shared__ float q_s[DEC_MAX_DIM], k_s[DEC_MAX_DIM];
  __shared__ float4 part[DEC_ROWS][DEC_TX];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, tx = tid % DEC_TX, ty = tid / DEC_TX;
  const int entry = blockIdx.z, head = blockIdx.y, col = blockIdx.x * DEC_COLS + tx * 4;
  const size_t row = (size_t)entry * proj_stride;
  const bool live = col < vdim;                           // vdim is a multiple of 4
  float4* S = reinterpret_cast<float4*>(state + (size_t)state_slots[entry] * slot_stride + (size_t)head * dim * vdim + col);
  const int pitch = vdim / 4;
  float4 s[DEC_BATCH];
  auto load = [&](int r0) {
#pragma unroll
    for (int i = 0; i < DEC_BATCH; ++i) {
      const int r = r0 + ty + i * DEC_ROWS;
      if (live && r < dim) s[i] = S[(size_t)r * pitch];
    }
  };
  load(0);                                                // under the sums and the activations below
  for (int d = tid; d < dim; d += DEC_THREADS) {
    q_s[d] = silu_f(proj.at(row + (size_t)head * dim + d));
    k_s[d] = silu_f(proj.at(row + (size_t)(heads + head) * dim + d));
  }
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  if (live)
#pragma unroll
    for (int c = 0; c < 4; ++c) v[c] = silu_f(proj.at(row + (size_t)2 * heads * dim + (size_t)head * vdim + col + c));
  const float d = decay[head];
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  __syncthreads();
  for (int r0 = 0; r0 < dim; r0 += DEC_BATCH * DEC_ROWS) {
    if (r0) load(r0);
#pragma unroll
    for (int i = 0; i < DEC_BATCH; ++i) {
      const int r = r0 + ty + i * DEC_ROWS;
      if (!live || r >= dim) continue;
      const float kr = k_s[r], qr = q_s[r];
      s[i].x = fmaf(d, s[i].x, kr * v[0]); s[i].y = fmaf(d, s[i].y, kr * v[1]);
      s[i].z = fmaf(d, s[i].z, kr * v[2]); s[i].w = fmaf(d, s[i].w, kr * v[3]);
      o[0] = fmaf(s[i].x, qr, o[0]); o[1] = fmaf(s[i].y, qr, o[1]);
      o[2] = fmaf(s[i].z, qr, o[2]); o[3] = fmaf(s[i].w, qr, o[3]);
      S[(size_t)r * pitch] = s[i];
    }
  }
  part[ty][tx] = make_float4(o[0], o[1], o[2], o[3]);
  __syncthreads();
  if (ty == 0 && live) {
    float4 a = part[0][tx];
#pragma unroll
    for (int g = 1; g < DEC_ROWS; ++g) {
      const float4 b = part[g][tx];
      a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w;
    }
    float* dst = out + (size_t)entry * out_stride + (size_t)head * vdim + col;
    dst[0] = a.x; dst[1] = a.y; dst[2] = a.z; dst[3] = a.w;
  }
}

// ---- prompt portions -----------------------------------------------------------------------------------------
constexpr int CC = 64, VT = 64, WARPS = 8, THREADS = WARPS * 32, PAD = 8, VP = VT + PAD;
constexpr int HALF = VT / 2;          // a warp of chunk_out makes 16 tokens x HALF columns, one of chunk_state 16 rows x HALF columns
using bf16 = __nv_bfloat16;

// The chunk with the running number idx: its entry, first token, length and place among its entry's chunks; false when the
// step has fewer chunks.
__device__ __forceinline__ bool chunk_of(const int* cu_tokens, int n_entries, int idx, int& c0, int& n) {
  for (int e = 0; e < n_entries; ++e) {
    const int t0 = cu_tokens[e], len = cu_tokens[e + 1] - t0, chunks = (len + CC - 1) / CC;
    if (idx < chunks) { c0 = t0 + idx * CC; n = min(CC, len - idx * CC); return true; }
    idx -= chunks;
  }
  return false;
}

// seg[chunk, head] [dim, vdim] = sum_j d^(n-1-j) k_j v_j^T.  Grid (chunks, heads, value tiles).
__global__ void __launch_bounds__(THREADS)
lightning_chunk_state_kernel(const bf16* __restrict__ k, const bf16* __restrict__ v, long long stride, const float* __restrict__ decay,
                             const int* __restrict__ cu_tokens, int n_entries, int heads, int dim, int vdim, float* __restrict__ seg) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ float pw[CC];
  pdl_launch_dependents();
  pdl_wait();
  int c0, n;
  if (!chunk_of(cu_tokens, n_entries, blockIdx.x, c0, n)) return;
  const int head = blockIdx.y, col0 = blockIdx.z * VT, kp = dim + PAD;
  bf16* k_s = reinterpret_cast<bf16*>(smem_raw);          // [CC][dim + PAD]
  bf16* v_s = k_s + CC * kp;                              // [3][CC][VP]: the decayed values in three pieces
  bring_rows<CC, THREADS>(k_s, kp, k + (size_t)c0 * stride + (size_t)head * dim, stride, n, dim, dim);
  // a thread's eight-column pieces of the values: requested first, scaled and split when the powers of the decay are there
  constexpr int PIECES = CC * (VT / 8) / THREADS;
  const bf16* src = v + (size_t)c0 * stride + (size_t)head * vdim + col0;
  float x[PIECES][8];
#pragma unroll
  for (int p = 0; p < PIECES; ++p) {
    const int i = threadIdx.x + p * THREADS, r = i / (VT / 8), c = (i % (VT / 8)) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) x[p][j] = 0.f;
    if (r < n && col0 + c < vdim) Vec8<bf16>::load(src + (size_t)r * stride + c, x[p]);
  }
  if (threadIdx.x < CC) pw[threadIdx.x] = powf(decay[head], (float)threadIdx.x);
  __syncthreads();
#pragma unroll
  for (int p = 0; p < PIECES; ++p) {
    const int i = threadIdx.x + p * THREADS, r = i / (VT / 8), c = (i % (VT / 8)) * 8;
    const float w = r < n ? pw[n - 1 - r] : 0.f;
    uint32_t q[4][3];
#pragma unroll
    for (int j = 0; j < 4; ++j) split3(x[p][2 * j] * w, x[p][2 * j + 1] * w, q[j]);
#pragma unroll
    for (int s = 0; s < 3; ++s)
      *reinterpret_cast<uint4*>(v_s + (s * CC + r) * VP + c) = make_uint4(q[0][s], q[1][s], q[2][s], q[3][s]);
  }
  cp_async_wait_all();
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, half = (warp & 1) * HALF;
  float* dst = seg + ((size_t)blockIdx.x * heads + head) * dim * vdim;
  // a warp makes two tiles of 16 rows x HALF columns at a time, so that a piece of the values it loads serves both
  for (int m0 = (warp >> 1) * 32; m0 < dim; m0 += WARPS / 2 * 32) {
    const bool two = m0 + 16 < dim;
    float acc[2][HALF / 8][4];
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int i = 0; i < HALF / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[h][i][j] = 0.f;
#pragma unroll
    for (int t0 = 0; t0 < CC; t0 += 16) {
      uint32_t a[2][4];
      const bf16* at = k_s + (t0 + (lane & 7) + ((lane >> 4) << 3)) * kp + m0 + (((lane >> 3) & 1) << 3);
      ldsm4_t(a[0], at);
      ldsm4_t(a[1], two ? at + 16 : at);
#pragma unroll
      for (int s = 0; s < 3; ++s)
#pragma unroll
        for (int i = 0; i < HALF / 16; ++i) {
          uint32_t b[4];
          ldsm4_t(b, v_s + (s * CC + t0 + (lane & 15)) * VP + half + i * 16 + ((lane >> 4) << 3));
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            mma(acc[h][2 * i], a[h], b[0], b[1]);
            mma(acc[h][2 * i + 1], a[h], b[2], b[3]);
          }
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      if (h && !two) break;
      const int r = m0 + 16 * h + (lane >> 2);
#pragma unroll
      for (int i = 0; i < HALF / 8; ++i) {
        const int c = col0 + half + i * 8 + 2 * (lane & 3);
        if (c >= vdim) continue;
        *reinterpret_cast<float2*>(dst + (size_t)r * vdim + c) = make_float2(acc[h][i][0], acc[h][i][1]);
        *reinterpret_cast<float2*>(dst + (size_t)(r + 8) * vdim + c) = make_float2(acc[h][i][2], acc[h][i][3]);
      }
    }
  }
}

// seg[chunk] holds the chunk's own contribution on entry and the state that enters the chunk on exit; the request's state
// moves to the end of the entry.  A thread per two elements of the state; sixteen chunks' loads are issued together.
constexpr int CHAIN = 16;

__global__ void __launch_bounds__(256)
lightning_chunk_chain_kernel(float* __restrict__ seg, const float* __restrict__ decay, float* __restrict__ state, long long slot_stride,
                             const int* __restrict__ state_slots, const int* __restrict__ cu_tokens, int heads, int dim, int vdim) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t per = (size_t)heads * dim * vdim / 2;
  const size_t el = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (el >= per) return;
  const int entry = blockIdx.y;
  size_t first = 0;
  for (int e = 0; e < entry; ++e) first += (cu_tokens[e + 1] - cu_tokens[e] + CC - 1) / CC;
  const int len = cu_tokens[entry + 1] - cu_tokens[entry], chunks = (len + CC - 1) / CC;
  const float d = decay[el / ((size_t)dim * vdim / 2)];
  const float whole = powf(d, (float)CC), last = powf(d, (float)(len - (chunks - 1) * CC));
  float2* S_g = reinterpret_cast<float2*>(state + (size_t)state_slots[entry] * slot_stride) + el;
  float2* at = reinterpret_cast<float2*>(seg) + first * per + el;
  float2 S = *S_g;
  for (int c0 = 0; c0 < chunks; c0 += CHAIN) {
    float2 own[CHAIN];
#pragma unroll
    for (int i = 0; i < CHAIN; ++i)
      if (c0 + i < chunks) own[i] = at[(size_t)(c0 + i) * per];
#pragma unroll
    for (int i = 0; i < CHAIN; ++i) {
      if (c0 + i >= chunks) break;
      at[(size_t)(c0 + i) * per] = S;
      const float w = c0 + i + 1 < chunks ? whole : last;
      S.x = fmaf(w, S.x, own[i].x); S.y = fmaf(w, S.y, own[i].y);
    }
  }
  *S_g = S;
}

// The outputs of a chunk: two warps per 16 tokens, each half of the columns.  Grid (chunks, heads, value tiles).  KD > 0: the
// warp keeps its queries in registers (dim = 16 KD); 0: it reads them again where it needs them.
template <int KD>
__global__ void __launch_bounds__(THREADS)
lightning_chunk_out_kernel(float* __restrict__ out, long long out_stride, const bf16* __restrict__ q, const bf16* __restrict__ k,
                           const bf16* __restrict__ v, long long stride, const float* __restrict__ decay,
                           const int* __restrict__ cu_tokens, int n_entries, int heads, int dim, int vdim,
                           const float* __restrict__ seg) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ float pw[CC + 1];
  pdl_launch_dependents();
  pdl_wait();
  int c0, n;
  if (!chunk_of(cu_tokens, n_entries, blockIdx.x, c0, n)) return;
  const int head = blockIdx.y, col0 = blockIdx.z * VT, kp = dim + PAD;
  bf16* q_s = reinterpret_cast<bf16*>(smem_raw);          // [CC][dim + PAD]
  bf16* k_s = q_s + CC * kp;                              // [CC][dim + PAD]
  bf16* v_s = k_s + CC * kp;                              // [CC][VP]
  bf16* S_s = v_s + CC * VP;                              // [3][dim][VP]: the state that enters the chunk in three pieces
  // the state first (its pieces are made in registers), four eight-column pieces a thread in flight
  constexpr int BATCH = 4;
  const float* src = seg + ((size_t)blockIdx.x * heads + head) * dim * vdim + col0;
  float x[BATCH][8];
  auto fetch = [&](int i0) {
#pragma unroll
    for (int p = 0; p < BATCH; ++p) {
      const int i = i0 + threadIdx.x + p * THREADS, r = i / (VT / 8), c = (i % (VT / 8)) * 8;
      if (r < dim && col0 + c < vdim) Vec8<float>::load(src + (size_t)r * vdim + c, x[p]);
      else
#pragma unroll
        for (int j = 0; j < 8; ++j) x[p][j] = 0.f;
    }
  };
  fetch(0);
  bring_rows<CC, THREADS>(q_s, kp, q + (size_t)c0 * stride + (size_t)head * dim, stride, n, dim, dim);
  bring_rows<CC, THREADS>(k_s, kp, k + (size_t)c0 * stride + (size_t)head * dim, stride, n, dim, dim);
  bring_rows<CC, THREADS>(v_s, VP, v + (size_t)c0 * stride + (size_t)head * vdim + col0, stride, n, min(VT, vdim - col0), VT);
  if (threadIdx.x <= CC) pw[threadIdx.x] = powf(decay[head], (float)threadIdx.x);
  for (int i0 = 0; i0 < dim * (VT / 8); i0 += BATCH * THREADS) {
    if (i0) fetch(i0);
#pragma unroll
    for (int p = 0; p < BATCH; ++p) {
      const int i = i0 + threadIdx.x + p * THREADS, r = i / (VT / 8), c = (i % (VT / 8)) * 8;
      if (r >= dim) continue;
      uint32_t w[4][3];
#pragma unroll
      for (int j = 0; j < 4; ++j) split3(x[p][2 * j], x[p][2 * j + 1], w[j]);
#pragma unroll
      for (int s = 0; s < 3; ++s)
        *reinterpret_cast<uint4*>(S_s + (s * dim + r) * VP + c) = make_uint4(w[0][s], w[1][s], w[2][s], w[3][s]);
    }
  }
  cp_async_wait_all();
  __syncthreads();
  const int lane = threadIdx.x & 31, i0 = (threadIdx.x >> 6) * 16, half = ((threadIdx.x >> 5) & 1) * HALF;
  if (i0 >= n) return;
  const bf16* q_at = q_s + (i0 + (lane & 15)) * kp + ((lane >> 4) << 3);
  const int kd = KD > 0 ? KD : dim / 16;
  uint32_t qr[KD > 0 ? KD : 1][4];
  if constexpr (KD > 0) {
#pragma unroll
    for (int x = 0; x < KD; ++x) ldsm4(qr[x], q_at + 16 * x);
  }
  auto query = [&](int x, uint32_t (&a)[4]) {
    if constexpr (KD > 0) { a[0] = qr[x][0]; a[1] = qr[x][1]; a[2] = qr[x][2]; a[3] = qr[x][3]; }
    else ldsm4(a, q_at + 16 * x);
  };
  float o[HALF / 8][4];
#pragma unroll
  for (int i = 0; i < HALF / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
  // what the state that enters the chunk contributes: d^(i+1) S_0^T q_i
#pragma unroll KD > 0 ? KD : 2
  for (int x = 0; x < kd; ++x) {
    const int k0 = 16 * x;
    uint32_t a[4];
    query(x, a);
#pragma unroll
    for (int s = 0; s < 3; ++s)
#pragma unroll
      for (int i = 0; i < HALF / 16; ++i) {
        uint32_t b[4];
        ldsm4_t(b, S_s + (s * dim + k0 + (lane & 15)) * VP + half + i * 16 + ((lane >> 4) << 3));
        mma(o[2 * i], a, b[0], b[1]);
        mma(o[2 * i + 1], a, b[2], b[3]);
      }
  }
  const int ra = i0 + (lane >> 2), rb = ra + 8;           // the lane's two rows
#pragma unroll
  for (int i = 0; i < HALF / 8; ++i) {
    o[i][0] *= pw[ra + 1]; o[i][1] *= pw[ra + 1];
    o[i][2] *= pw[rb + 1]; o[i][3] *= pw[rb + 1];
  }
  // the chunk's own tokens, 16 keys at a time up to the warp's last row
  for (int j0 = 0; j0 <= i0; j0 += 16) {
    float p[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll KD > 0 ? KD : 4
    for (int x = 0; x < kd; ++x) {
      const int k0 = 16 * x;
      uint32_t a[4], b[4];
      query(x, a);
      ldsm4(b, k_s + (j0 + (lane & 7) + ((lane >> 4) << 3)) * kp + k0 + (((lane >> 3) & 1) << 3));
      mma(p[0], a, b[0], b[1]);
      mma(p[1], a, b[2], b[3]);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int dist = (c < 2 ? ra : rb) - (j0 + 8 * i + 2 * (lane & 3) + (c & 1));
        p[i][c] = dist >= 0 ? p[i][c] * pw[dist] : 0.f;
      }
    uint32_t w[4][3];
    split3(p[0][0], p[0][1], w[0]);
    split3(p[0][2], p[0][3], w[1]);
    split3(p[1][0], p[1][1], w[2]);
    split3(p[1][2], p[1][3], w[3]);
#pragma unroll
    for (int i = 0; i < HALF / 16; ++i) {
      uint32_t b[4];
      ldsm4_t(b, v_s + (j0 + (lane & 15)) * VP + half + i * 16 + ((lane >> 4) << 3));
#pragma unroll
      for (int s = 0; s < 3; ++s) {
        const uint32_t a[4] = {w[0][s], w[1][s], w[2][s], w[3][s]};
        mma(o[2 * i], a, b[0], b[1]);
        mma(o[2 * i + 1], a, b[2], b[3]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < HALF / 8; ++i) {
    const int c = col0 + half + i * 8 + 2 * (lane & 3);
    if (c >= vdim) continue;
    float* dst = out + (size_t)head * vdim + c;
    if (ra < n) *reinterpret_cast<float2*>(dst + (size_t)(c0 + ra) * out_stride) = make_float2(o[i][0], o[i][1]);
    if (rb < n) *reinterpret_cast<float2*>(dst + (size_t)(c0 + rb) * out_stride) = make_float2(o[i][2], o[i][3]);
  }
}

}  // namespace

// One token per entry.  proj: rows [q | k | v | ...] of the element kind, or float32 partial results [splits][rows][stride]; silu
// is taken here.  state: slot s at state + s * slot_stride, [heads, dim, vdim] float32; vdim a multiple of 4, dim up to 512.
LLMK_API int llmk_lightning_decode(float* out, long long out_stride, const void* proj, const float* partials, int splits,
                                   long long split_stride, long long proj_stride, const float* decay, float* state,
                                   long long slot_stride, const int* state_slots, int n_entries, int heads, int dim, int vdim,
                                   int dtype, cudaStream_t stream) {
  if (n_entries == 0) return 0;
  LLMK_REQUIRE((proj != nullptr) != (partials != nullptr), "lightning_decode: give proj or partials");
  LLMK_REQUIRE(dim > 0 && dim <= DEC_MAX_DIM && vdim > 0 && vdim % 4 == 0, "lightning_decode: key size %d (1 to %d) or value size %d (a multiple of 4)",
               dim, DEC_MAX_DIM, vdim);
  LLMK_REQUIRE(slot_stride % 4 == 0 && (uintptr_t)state % 16 == 0, "lightning_decode: the state must lie on the 16-byte grid");
  LLMK_REQUIRE(n_entries <= 65535 && heads <= 65535, "lightning_decode: too many entries or heads for one launch");
  return dispatch_dtype(dtype, [&](auto* tag) {
    using T = LLMK_ELEM(tag);
    MaybePartial<T> p{(const T*)proj, partials, splits, split_stride};
    launch_kernel(lightning_decode_kernel<T>, dim3((vdim + DEC_COLS - 1) / DEC_COLS, heads, n_entries), dim3(DEC_THREADS), 0, stream, out,
                  out_stride, p, proj_stride, decay, state, slot_stride, state_slots, heads, dim, vdim);
    LLMK_LAUNCH_CHECK("lightning_decode");
  });
}

// Entries of any length, bfloat16 q, k, v with silu already taken (one row stride; head h at column h * dim, of v h * vdim).
// dim a multiple of 16 up to 256, vdim of 8.  seg: float32 scratch [n_tokens / 64 + n_entries, heads, dim, vdim].
LLMK_API int llmk_lightning_chunks(float* out, long long out_stride, const void* q, const void* k, const void* v, long long stride,
                                   const float* decay, float* state, long long slot_stride, const int* state_slots,
                                   const int* cu_tokens, int n_entries, int n_tokens, int heads, int dim, int vdim, float* seg,
                                   cudaStream_t stream) {
  if (n_entries == 0 || n_tokens == 0) return 0;
  LLMK_REQUIRE(dim > 0 && dim % 16 == 0 && dim <= 256 && vdim > 0 && vdim % 8 == 0,
               "lightning_chunks: key size %d (a multiple of 16 up to 256) or value size %d (a multiple of 8)", dim, vdim);
  LLMK_REQUIRE(stride % 8 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)k % 16 == 0 && (uintptr_t)v % 16 == 0 && out_stride % 2 == 0 &&
                   (uintptr_t)out % 8 == 0 && slot_stride % 4 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)seg % 16 == 0,
               "lightning_chunks: operands off the 16-byte grid");
  LLMK_REQUIRE(n_entries <= 65535 && heads <= 65535, "lightning_chunks: too many entries or heads for one launch");
  const int chunks = n_tokens / CC + n_entries, tiles = (vdim + VT - 1) / VT;
  const size_t smem1 = ((size_t)CC * (dim + PAD) + 3 * CC * VP) * sizeof(bf16);
  const size_t smem3 = ((size_t)2 * CC * (dim + PAD) + CC * VP + (size_t)3 * dim * VP) * sizeof(bf16);
  cudaFuncSetAttribute(lightning_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
  auto outputs = dim == 128 ? lightning_chunk_out_kernel<8> : dim == 64 ? lightning_chunk_out_kernel<4>
               : dim == 32 ? lightning_chunk_out_kernel<2> : lightning_chunk_out_kernel<0>;
  cudaFuncSetAttribute(outputs, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3);
  launch_kernel(lightning_chunk_state_kernel, dim3(chunks, heads, tiles), dim3(THREADS), smem1, stream, (const bf16*)k, (const bf16*)v, stride,
                decay, cu_tokens, n_entries, heads, dim, vdim, seg);
  const size_t per = (size_t)heads * dim * vdim / 2;
  launch_kernel(lightning_chunk_chain_kernel, dim3((unsigned)((per + 255) / 256), n_entries), dim3(256), 0, stream, seg, decay, state,
                slot_stride, state_slots, cu_tokens, heads, dim, vdim);
  launch_kernel(outputs, dim3(chunks, heads, tiles), dim3(THREADS), smem3, stream, out, out_stride, (const bf16*)q,
                (const bf16*)k, (const bf16*)v, stride, decay, cu_tokens, n_entries, heads, dim, vdim, (const float*)seg);
  LLMK_LAUNCH_CHECK("lightning_chunks");
}
