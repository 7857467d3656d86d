// Matrix memory with exponential gates (mLSTM).  Per head, with a log input gate i and a log forget gate f <= 0 a token:
//
//   i = cap tanh((z_i + b_i) / cap),   f = logsigmoid(cap tanh((z_f + b_f) / cap))
//   m_t = max(f + m_(t-1), i)                                          the running maximum, 0 at the start
//   S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k_t v_t^T      S [dim, vdim]
//   n_t = exp(f + m_(t-1) - m_t) n_(t-1) + exp(i - m_t) k_t            n [dim]
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)             q_t scaled by q_scale
//
// S, n and m are float32 and live in the request's state slot (zero at admission): [S: heads * dim * vdim | n: heads * blocks *
// dim | m: heads * blocks], each from a multiple of 4 floats on.  A CTA of the kernels that walk token by token owns COLS value
// columns of a head and needs n and m as well; so that no CTA reads what another one renews, n and m are kept once per block of
// COLS columns (blocks = vdim / COLS, rounded up), all copies alike.  Gates, states and sums are float32.
//
// Three forms, by what a step brings:
//   mlstm_decode   single tokens: the state is read and written once, everything else is small (as in lightning.cu).
//   mlstm_scan     token by token for any sizes: float32, short portions, sizes off the grid.
//   mlstm_chunks   prompt portions in bfloat16, chunks of 64 tokens.  With b_t the running sum of f over the chunk, g_t = i_t - b_t,
//                  and S_0, n_0, m_0 what enters the chunk,
//                      m_t = b_t + max(m_0, max_{j <= t} g_j)
//                      S_t = exp(b_t + m_0 - m_t) S_0 + sum_{j <= t} exp(g_j + b_t - m_t) k_j v_j^T        n_t alike
//                  every exponent is at most zero.  The chunks' own sums are made side by side, relative to the chunk's own
//                  maximum M = b_n + max_j g_j (chunk_state), chained from the request's state (chunk_chain: F = b_n,
//                  m' = max(F + m, M), S' = exp(F + m - m') S + exp(M - m') E), and the outputs are made side by side
//                  (chunk_out).  q, k, v are bfloat16, so their products have exact factors; float32 operands of a product (the
//                  state, the weighted scores, the weighted values) enter it as three bfloat16 numbers, which hold their 24
//                  bits, and every sum is float32.  The products are warp-level MMAs, laid out as in lightning.cu.
#include "warp_mma.cuh"

namespace {

constexpr int COLS = 64;
constexpr float DENOM_EPS = 1e-6f;

__device__ __forceinline__ float log_sigmoid(float x) { return x >= 0.f ? -log1pf(expf(-x)) : x - log1pf(expf(x)); }
__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }

struct Gates {
  const float *i_bias, *f_bias;         // [heads]
  float cap, q_scale;
};
struct State {
  float* base; long long slot_stride, n_off, m_off;      // element offsets of n and m within a slot
  const int* slots;
};

// ---- single tokens -----------------------------------------------------------------------------------------
constexpr int DEC_TX = COLS / 4, DEC_ROWS = 8, DEC_THREADS = DEC_TX * DEC_ROWS, DEC_BATCH = 16, DEC_MAX_DIM = 512;

// proj row e: [q: heads * dim | k: heads * dim | v: heads * vdim | .. | at gate_col: i: heads | f: heads].  What the CTA needs of it
// is summed into shared memory first, every load of the partial results in flight at once (VEC: four columns a thread; dim and
// proj_stride on the 4-grid), under the loads of the state's first rows.
template <bool VEC>
__global__ void __launch_bounds__(DEC_THREADS)
mlstm_decode_kernel(float* __restrict__ out, long long out_stride, MaybePartial<float> proj, long long proj_stride, long long gate_col,
                    Gates gt, State st, int heads, int dim, int vdim) {
  __shared__ __align__(16) float q_s[DEC_MAX_DIM], k_s[DEC_MAX_DIM], v_s[COLS], z_s[2];
  __shared__ float4 part[DEC_ROWS][DEC_TX];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, tx = tid % DEC_TX, ty = tid / DEC_TX;
  const int entry = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * COLS, col = col0 + tx * 4;
  const size_t row = (size_t)entry * proj_stride;
  const bool live = col < vdim;                           // vdim is a multiple of 4
  float* slot = st.base + (size_t)st.slots[entry] * st.slot_stride;
  float4* S = reinterpret_cast<float4*>(slot + (size_t)head * dim * vdim + col);
  const size_t copy = (size_t)head * gridDim.x + blockIdx.x;
  float *n_g = slot + st.n_off + copy * dim, *m_g = slot + st.m_off + copy;
  const int pitch = vdim / 4;
  float4 s[DEC_BATCH];
  auto load = [&](int r0) {
#pragma unroll
    for (int i = 0; i < DEC_BATCH; ++i) {
      const int r = r0 + ty + i * DEC_ROWS;
      if (live && r < dim) s[i] = S[(size_t)r * pitch];
    }
  };
  load(0);
  const float m_old = *m_g;
  const size_t q0 = row + (size_t)head * dim, k0 = row + (size_t)(heads + head) * dim, v0 = row + (size_t)2 * heads * dim + (size_t)head * vdim + col0;
  const int cols = min(COLS, vdim - col0);
  constexpr int N = VEC ? 4 : 1;
  // from the last thread down, so that the two gates' sums run beside the vectors'
  if (tid >= DEC_THREADS - 2) z_s[tid - (DEC_THREADS - 2)] = proj.at(row + gate_col + (tid - (DEC_THREADS - 2)) * heads + head);
  for (int i = tid; i < (2 * dim + cols) / N; i += DEC_THREADS) {
    const int e = i * N;
    float* dst = e < dim ? q_s + e : e < 2 * dim ? k_s + e - dim : v_s + e - 2 * dim;
    const size_t src = e < dim ? q0 + e : e < 2 * dim ? k0 + e - dim : v0 + e - 2 * dim;
    if constexpr (VEC) {
      float v[4];
      proj.at4(src, v);
      *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
      *dst = proj.at(src);
    }
  }
  __syncthreads();
  const float gi = soft_cap(z_s[0] + gt.i_bias[head], gt.cap), gf = log_sigmoid(soft_cap(z_s[1] + gt.f_bias[head], gt.cap));
  const float m = fmaxf(gf + m_old, gi), keep = expf(gf + m_old - m), write = expf(gi - m);
  float nq = 0.f;
  for (int d = tid; d < dim; d += DEC_THREADS) {
    const float nd = fmaf(keep, n_g[d], k_s[d] * write);
    n_g[d] = nd;
    nq = fmaf(nd, q_s[d], nq);
  }
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  if (live) {
    const float4 v4 = *reinterpret_cast<const float4*>(v_s + 4 * tx);
    v[0] = v4.x * write; v[1] = v4.y * write; v[2] = v4.z * write; v[3] = v4.w * write;
  }
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  for (int r0 = 0; r0 < dim; r0 += DEC_BATCH * DEC_ROWS) {
    if (r0) load(r0);
#pragma unroll
    for (int i = 0; i < DEC_BATCH; ++i) {
      const int r = r0 + ty + i * DEC_ROWS;
      if (!live || r >= dim) continue;
      const float kr = k_s[r], qr = q_s[r];
      s[i].x = fmaf(keep, s[i].x, kr * v[0]); s[i].y = fmaf(keep, s[i].y, kr * v[1]);
      s[i].z = fmaf(keep, s[i].z, kr * v[2]); s[i].w = fmaf(keep, s[i].w, kr * v[3]);
      o[0] = fmaf(s[i].x, qr, o[0]); o[1] = fmaf(s[i].y, qr, o[1]);
      o[2] = fmaf(s[i].z, qr, o[2]); o[3] = fmaf(s[i].w, qr, o[3]);
      S[(size_t)r * pitch] = s[i];
    }
  }
  part[ty][tx] = make_float4(o[0], o[1], o[2], o[3]);
  nq = block_sum(nq, red) * gt.q_scale;                   // its barriers also stand between part and its readers
  if (tid == 0) *m_g = m;                                 // every thread has read the old one
  if (ty == 0 && live) {
    float4 a = part[0][tx];
#pragma unroll
    for (int g = 1; g < DEC_ROWS; ++g) {
      const float4 b = part[g][tx];
      a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w;
    }
    const float f = gt.q_scale / (fmaxf(fabsf(nq), expf(-m)) + DENOM_EPS);
    float* dst = out + (size_t)entry * out_stride + (size_t)head * vdim + col;
    dst[0] = a.x * f; dst[1] = a.y * f; dst[2] = a.z * f; dst[3] = a.w * f;
  }
}

// ---- token by token -----------------------------------------------------------------------------------------
// Thread (j, g) keeps the 8 x 4 block of S at rows 8 g .., columns 4 j .. and the 8 rows of n; tokens are staged SC at a time.
constexpr int ROWS = 8, SC = 8, TX = COLS / 4, MAX_GROUPS = 32;

__global__ void __launch_bounds__(TX * MAX_GROUPS)
mlstm_scan_kernel(float* __restrict__ out, long long out_stride, const float* __restrict__ proj, long long proj_stride,
                  long long gate_col, Gates gt, State st, const int* __restrict__ cu_tokens, int heads, int dim, int vdim) {
  extern __shared__ __align__(16) float smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int groups = blockDim.y, dpad = groups * ROWS;
  float* q_s = smem;                          // [SC][dpad]
  float* k_s = q_s + SC * dpad;               // [SC][dpad]: keys times the input gate
  float* v_s = k_s + SC * dpad;               // [SC][COLS]
  float* part = v_s + SC * COLS;              // [SC][groups][COLS]
  float* nq_s = part + SC * groups * COLS;    // [SC][groups]
  float* g_s = nq_s + SC * groups;            // [SC] i, then the write factor; [SC] f, then the keep factor; [SC] the floor of |n.q|
  const int j = threadIdx.x, g = threadIdx.y, tid = g * TX + j, nthreads = TX * groups;
  const int entry = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * COLS + 4 * j;
  const int t0 = cu_tokens[entry], t1 = cu_tokens[entry + 1];
  if (t0 >= t1) return;
  float* slot = st.base + (size_t)st.slots[entry] * st.slot_stride;
  float* S_g = slot + (size_t)head * dim * vdim;
  const size_t copy = (size_t)head * gridDim.x + blockIdx.x;
  float *n_g = slot + st.n_off + copy * dim, *m_g = slot + st.m_off + copy;
  float S[ROWS][4], N[ROWS];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int d = g * ROWS + r;
    N[r] = d < dim ? n_g[d] : 0.f;
#pragma unroll
    for (int c = 0; c < 4; ++c) S[r][c] = (d < dim && col0 + c < vdim) ? S_g[(size_t)d * vdim + col0 + c] : 0.f;
  }
  float m = *m_g;                             // carried by thread 0
  for (int c0 = t0; c0 < t1; c0 += SC) {
    const int n = min(SC, t1 - c0);
    __syncthreads();
    if (tid < n) {
      const float* p = proj + (size_t)(c0 + tid) * proj_stride + gate_col;
      g_s[tid] = soft_cap(p[head] + gt.i_bias[head], gt.cap);
      g_s[SC + tid] = log_sigmoid(soft_cap(p[heads + head] + gt.f_bias[head], gt.cap));
    }
    __syncthreads();
    if (tid == 0) {
      for (int c = 0; c < n; ++c) {
        const float gi = g_s[c], gf = g_s[SC + c], mn = fmaxf(gf + m, gi);
        g_s[c] = expf(gi - mn);
        g_s[SC + c] = expf(gf + m - mn);
        g_s[2 * SC + c] = expf(-mn);
        m = mn;
      }
    }
    __syncthreads();
    for (int i = tid; i < n * dpad; i += nthreads) {
      const int c = i / dpad, d = i % dpad;
      const float* p = proj + (size_t)(c0 + c) * proj_stride;
      q_s[i] = d < dim ? p[(size_t)head * dim + d] * gt.q_scale : 0.f;
      k_s[i] = d < dim ? p[(size_t)(heads + head) * dim + d] * g_s[c] : 0.f;
    }
    for (int i = tid; i < n * COLS; i += nthreads) {
      const int c = i / COLS, cc = blockIdx.x * COLS + i % COLS;
      v_s[i] = cc < vdim ? proj[(size_t)(c0 + c) * proj_stride + (size_t)2 * heads * dim + (size_t)head * vdim + cc] : 0.f;
    }
    __syncthreads();
    for (int c = 0; c < n; ++c) {
      const float4 v4 = *reinterpret_cast<const float4*>(v_s + c * COLS + 4 * j);
      const float vv[4] = {v4.x, v4.y, v4.z, v4.w};
      const float keep = g_s[SC + c];
      float o[4] = {0.f, 0.f, 0.f, 0.f}, nq = 0.f;
#pragma unroll
      for (int r = 0; r < ROWS; r += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(k_s + c * dpad + g * ROWS + r);
        const float4 q4 = *reinterpret_cast<const float4*>(q_s + c * dpad + g * ROWS + r);
        const float kr[4] = {k4.x, k4.y, k4.z, k4.w}, qr[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          N[r + x] = fmaf(keep, N[r + x], kr[x]);
          nq = fmaf(N[r + x], qr[x], nq);
#pragma unroll
          for (int cc = 0; cc < 4; ++cc) {
            S[r + x][cc] = fmaf(keep, S[r + x][cc], kr[x] * vv[cc]);
            o[cc] = fmaf(S[r + x][cc], qr[x], o[cc]);
          }
        }
      }
      *reinterpret_cast<float4*>(part + (c * groups + g) * COLS + 4 * j) = make_float4(o[0], o[1], o[2], o[3]);
      if (j == 0) nq_s[c * groups + g] = nq;
    }
    __syncthreads();
    for (int i = tid; i < n * COLS; i += nthreads) {
      const int c = i / COLS, jj = i % COLS, cc = blockIdx.x * COLS + jj;
      if (cc >= vdim) continue;
      float o = 0.f, nq = 0.f;
      for (int gg = 0; gg < groups; ++gg) { o += part[(c * groups + gg) * COLS + jj]; nq += nq_s[c * groups + gg]; }
      out[(size_t)(c0 + c) * out_stride + (size_t)head * vdim + cc] = o / (fmaxf(fabsf(nq), g_s[2 * SC + c]) + DENOM_EPS);
    }
  }
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int d = g * ROWS + r;
    if (d >= dim) continue;
    if (j == 0) n_g[d] = N[r];
#pragma unroll
    for (int c = 0; c < 4; ++c)
      if (col0 + c < vdim) S_g[(size_t)d * vdim + col0 + c] = S[r][c];
  }
  if (tid == 0) *m_g = m;
}

// ---- prompt portions ------------------------------------------------------------------------------------------
constexpr int CC = 64, VT = COLS, WARPS = 8, THREADS = WARPS * 32, PAD = 8, VP = VT + PAD, HALF = VT / 2;
using bf16 = __nv_bfloat16;

struct Chunk { int entry, c0, n; bool last; };

// The chunk with the running number idx; false when the step has fewer chunks.
__device__ __forceinline__ bool chunk_of(const int* cu_tokens, int n_entries, int idx, Chunk& ch) {
  for (int e = 0; e < n_entries; ++e) {
    const int t0 = cu_tokens[e], len = cu_tokens[e + 1] - t0, chunks = (len + CC - 1) / CC;
    if (idx < chunks) { ch = {e, t0 + idx * CC, min(CC, len - idx * CC), idx + 1 == chunks}; return true; }
    idx -= chunks;
  }
  return false;
}

// One warp: b_s[t] = the running sum of f, g_s[t] = i_t - b_t, h_s[t] = max_{j <= t} g_j for the chunk's tokens (g is minus
// infinity and b stays behind the last one).  A lane holds two neighbouring tokens.
__device__ __forceinline__ void chunk_gates(const float* z, long long z_stride, const Gates& gt, int head, int heads, int c0, int n,
                                            float* b_s, float* g_s, float* h_s) {
  const int lane = threadIdx.x & 31;
  float gi[2], gf[2];
  const float ib = gt.i_bias[head], fb = gt.f_bias[head];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const float* p = z + (size_t)(c0 + min(2 * lane + x, n - 1)) * z_stride;
    gi[x] = p[head]; gf[x] = p[heads + head];
  }
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const bool on = 2 * lane + x < n;
    gi[x] = on ? soft_cap(gi[x] + ib, gt.cap) : -INFINITY;
    gf[x] = on ? log_sigmoid(soft_cap(gf[x] + fb, gt.cap)) : 0.f;
  }
  float sum = gf[0] + gf[1];
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, sum, o);
    if (lane >= o) sum += up;
  }
  const float b1 = sum, b0 = b1 - gf[1];
  const float g0 = gi[0] - b0, g1 = gi[1] - b1;
  float top = fmaxf(g0, g1);
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, top, o);
    if (lane >= o) top = fmaxf(top, up);
  }
  const float before = __shfl_up_sync(0xffffffffu, top, 1);
  b_s[2 * lane] = b0; b_s[2 * lane + 1] = b1;
  g_s[2 * lane] = g0; g_s[2 * lane + 1] = g1;
  h_s[2 * lane] = lane ? fmaxf(before, g0) : g0;
  h_s[2 * lane + 1] = top;
}

// Scratch of the chunks: per chunk and head E [dim, vdim] and e [dim] (the chunk's own sums, then the state that enters it),
// and four floats: F, M, and the maximum that enters the chunk.
struct Scratch { float *E, *e, *fm; };

// Grid (chunks, heads, value tiles).
__global__ void __launch_bounds__(THREADS)
mlstm_chunk_state_kernel(const bf16* __restrict__ k, const bf16* __restrict__ v, long long stride, const float* __restrict__ z,
                         long long z_stride, Gates gt, const int* __restrict__ cu_tokens, int n_entries, int heads, int dim, int vdim,
                         Scratch sc) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ float b_s[CC], g_s[CC], h_s[CC], w_s[CC];
  pdl_launch_dependents();
  pdl_wait();
  Chunk ch;
  if (!chunk_of(cu_tokens, n_entries, blockIdx.x, ch)) return;
  const int c0 = ch.c0, n = ch.n;
  const int head = blockIdx.y, col0 = blockIdx.z * VT, kp = dim + PAD;
  const size_t unit = (size_t)blockIdx.x * heads + head;
  bf16* k_s = reinterpret_cast<bf16*>(smem_raw);          // [CC][dim + PAD]
  bf16* v_s = k_s + CC * kp;                              // [3][CC][VP]: the weighted values in three pieces
  bring_rows<CC, THREADS>(k_s, kp, k + (size_t)c0 * stride + (size_t)head * dim, stride, n, dim, dim);
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
  if (threadIdx.x < 32) {
    chunk_gates(z, z_stride, gt, head, heads, c0, n, b_s, g_s, h_s);
    __syncwarp();
    const float top = h_s[CC - 1];
#pragma unroll
    for (int y = 0; y < 2; ++y) w_s[2 * threadIdx.x + y] = expf(g_s[2 * threadIdx.x + y] - top);      // relative to the chunk's maximum
    if (threadIdx.x == 0 && blockIdx.z == 0) { sc.fm[unit * 4] = b_s[CC - 1]; sc.fm[unit * 4 + 1] = b_s[CC - 1] + top; }
  }
  __syncthreads();
#pragma unroll
  for (int p = 0; p < PIECES; ++p) {
    const int i = threadIdx.x + p * THREADS, r = i / (VT / 8), c = (i % (VT / 8)) * 8;
    const float w = w_s[r];
    uint32_t q[4][3];
#pragma unroll
    for (int j = 0; j < 4; ++j) split3(x[p][2 * j] * w, x[p][2 * j + 1] * w, q[j]);
#pragma unroll
    for (int s = 0; s < 3; ++s)
      *reinterpret_cast<uint4*>(v_s + (s * CC + r) * VP + c) = make_uint4(q[0][s], q[1][s], q[2][s], q[3][s]);
  }
  cp_async_wait_all();
  __syncthreads();
  if (blockIdx.z == 0)
    for (int d = threadIdx.x; d < dim; d += THREADS) {
      float a = 0.f;
#pragma unroll 8
      for (int t = 0; t < CC; ++t) a = fmaf(w_s[t], __bfloat162float(k_s[t * kp + d]), a);
      sc.e[unit * dim + d] = a;
    }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, half = (warp & 1) * HALF;
  float* dst = sc.E + unit * dim * vdim;
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

// E and e hold the chunk's own sums on entry and the state that enters the chunk on exit; S and n of the request's slot move to
// the entry's end.  m itself is renewed by chunk_out: here every thread reads it.  A thread per two elements of S or n.
constexpr int CHAIN = 8;

__global__ void __launch_bounds__(256)
mlstm_chunk_chain_kernel(Scratch sc, State st, const int* __restrict__ cu_tokens, int heads, int dim, int vdim, int blocks) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t per_S = (size_t)heads * dim * vdim / 2, per_n = (size_t)heads * dim / 2;
  const size_t el = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (el >= per_S + per_n) return;
  const bool is_n = el >= per_S;
  const size_t at0 = is_n ? el - per_S : el, per = is_n ? per_n : per_S;
  const int head = (int)(at0 / (is_n ? dim / 2 : (size_t)dim * vdim / 2));
  const int entry = blockIdx.y;
  size_t first = 0;
  for (int e = 0; e < entry; ++e) first += (cu_tokens[e + 1] - cu_tokens[e] + CC - 1) / CC;
  const int len = cu_tokens[entry + 1] - cu_tokens[entry], chunks = (len + CC - 1) / CC;
  if (chunks == 0) return;
  float* slot = st.base + (size_t)st.slots[entry] * st.slot_stride;
  float m = slot[st.m_off + (size_t)head * blocks];
  const size_t d2 = is_n ? at0 - (size_t)head * (dim / 2) : 0;      // n: the pair's place in its head
  float2* own_g = is_n ? reinterpret_cast<float2*>(slot + st.n_off + (size_t)head * blocks * dim) + d2 : reinterpret_cast<float2*>(slot) + at0;
  float2* at = reinterpret_cast<float2*>(is_n ? sc.e : sc.E) + first * per + at0;
  float* fm = sc.fm + (first * heads + head) * 4;
  const bool says = is_n && d2 == 0;
  float2 S = *own_g;
  for (int c0 = 0; c0 < chunks; c0 += CHAIN) {
    float2 own[CHAIN], f[CHAIN];
#pragma unroll
    for (int i = 0; i < CHAIN; ++i)
      if (c0 + i < chunks) {
        own[i] = at[(size_t)(c0 + i) * per];
        f[i] = *reinterpret_cast<const float2*>(fm + (size_t)(c0 + i) * heads * 4);
      }
#pragma unroll
    for (int i = 0; i < CHAIN; ++i) {
      if (c0 + i >= chunks) break;
      at[(size_t)(c0 + i) * per] = S;
      if (says) fm[(size_t)(c0 + i) * heads * 4 + 2] = m;
      const float mn = fmaxf(f[i].x + m, f[i].y), a = expf(f[i].x + m - mn), b = expf(f[i].y - mn);
      S.x = fmaf(a, S.x, b * own[i].x); S.y = fmaf(a, S.y, b * own[i].y);
      m = mn;
    }
  }
  *own_g = S;
  if (is_n)
    for (int b = 1; b < blocks; ++b) own_g[(size_t)b * (dim / 2)] = S;
}

// The outputs of a chunk: two warps per 16 tokens, each half of the columns.  Grid (chunks, heads, value tiles).  KD > 0: the
// warp keeps its queries in registers (dim = 16 KD); 0: it reads them again where it needs them.
template <int KD>
__global__ void __launch_bounds__(THREADS)
mlstm_chunk_out_kernel(float* __restrict__ out, long long out_stride, const bf16* __restrict__ q, const bf16* __restrict__ k,
                       const bf16* __restrict__ v, long long stride, const float* __restrict__ z, long long z_stride, Gates gt, State st,
                       const int* __restrict__ cu_tokens, int n_entries, int heads, int dim, int vdim, Scratch sc) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ float b_s[CC], g_s[CC], h_s[CC], m_s[CC], nq_s[CC];
  __shared__ __align__(8) float n_s[256];                 // n_0
  pdl_launch_dependents();
  pdl_wait();
  Chunk ch;
  if (!chunk_of(cu_tokens, n_entries, blockIdx.x, ch)) return;
  const int c0 = ch.c0, n = ch.n;
  const int head = blockIdx.y, col0 = blockIdx.z * VT, kp = dim + PAD;
  const size_t unit = (size_t)blockIdx.x * heads + head;
  bf16* q_s = reinterpret_cast<bf16*>(smem_raw);          // [CC][dim + PAD]
  bf16* k_s = q_s + CC * kp;                              // [CC][dim + PAD]
  bf16* v_s = k_s + CC * kp;                              // [CC][VP]
  bf16* S_s = v_s + CC * VP;                              // [3][dim][VP]: the state that enters the chunk in three pieces
  constexpr int BATCH = 4;
  const float* src = sc.E + unit * dim * vdim + col0;
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
  if (threadIdx.x < dim) n_s[threadIdx.x] = sc.e[unit * dim + threadIdx.x];
  const float m0 = sc.fm[unit * 4 + 2];
  if (threadIdx.x < 32) {
    chunk_gates(z, z_stride, gt, head, heads, c0, n, b_s, g_s, h_s);
    __syncwarp();
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int t = 2 * threadIdx.x + y;
      m_s[t] = b_s[t] + fmaxf(m0, h_s[t]);
    }
    __syncwarp();
    if (ch.last && threadIdx.x == 0)
      st.base[(size_t)st.slots[ch.entry] * st.slot_stride + st.m_off + (size_t)head * gridDim.z + blockIdx.z] = m_s[n - 1];
  }
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
  {                                                       // n_0 . q of every token: four threads a token
    const int t = threadIdx.x >> 2, l = threadIdx.x & 3;
    float a = 0.f;
#pragma unroll 4
    for (int d = 2 * l; d < dim; d += 8) {
      const float2 nv = *reinterpret_cast<const float2*>(n_s + d);
      const float2 qv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(q_s + t * kp + d));
      a = fmaf(nv.x, qv.x, a); a = fmaf(nv.y, qv.y, a);
    }
    a += __shfl_xor_sync(0xffffffffu, a, 1);
    a += __shfl_xor_sync(0xffffffffu, a, 2);
    if (l == 0) nq_s[t] = a;
  }
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
  // what the state that enters the chunk contributes: exp(b_t + m_0 - m_t) S_0^T q_t
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
  const float la = b_s[ra] - m_s[ra], lb = b_s[rb] - m_s[rb];
  const float ea = expf(la + m0) * gt.q_scale, eb = expf(lb + m0) * gt.q_scale;
#pragma unroll
  for (int i = 0; i < HALF / 8; ++i) {
    o[i][0] *= ea; o[i][1] *= ea;
    o[i][2] *= eb; o[i][3] *= eb;
  }
  float na = 0.f, nb = 0.f;                               // the rows' sums of weighted scores: n . q but for n_0's share
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
        const int j = j0 + 8 * i + 2 * (lane & 3) + (c & 1);
        const bool seen = j <= (c < 2 ? ra : rb);
        p[i][c] = seen ? p[i][c] * gt.q_scale * expf(g_s[j] + (c < 2 ? la : lb)) : 0.f;
        if (c < 2) na += p[i][c]; else nb += p[i][c];
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
  for (int x = 1; x < 4; x <<= 1) {                       // the four lanes that share the rows
    na += __shfl_xor_sync(0xffffffffu, na, x);
    nb += __shfl_xor_sync(0xffffffffu, nb, x);
  }
  const float da = 1.f / (fmaxf(fabsf(fmaf(ea, nq_s[ra], na)), expf(-m_s[ra])) + DENOM_EPS);
  const float db = 1.f / (fmaxf(fabsf(fmaf(eb, nq_s[rb], nb)), expf(-m_s[rb])) + DENOM_EPS);
#pragma unroll
  for (int i = 0; i < HALF / 8; ++i) {
    const int c = col0 + half + i * 8 + 2 * (lane & 3);
    if (c >= vdim) continue;
    float* dst = out + (size_t)head * vdim + c;
    if (ra < n) *reinterpret_cast<float2*>(dst + (size_t)(c0 + ra) * out_stride) = make_float2(o[i][0] * da, o[i][1] * da);
    if (rb < n) *reinterpret_cast<float2*>(dst + (size_t)(c0 + rb) * out_stride) = make_float2(o[i][2] * db, o[i][3] * db);
  }
}

}  // namespace

LLMK_API int llmk_mlstm_cols() { return COLS; }

// One token per entry (single != 0) or any entries token by token.  proj: float32 rows of proj_stride, [q | k | v | .. | i | f] with
// i at column gate_col, or (single only) the float32 partial results [splits][rows][proj_stride].  i_bias, f_bias float32
// [heads].  state: slot s at state + s * slot_stride, n and m at n_off and m_off within it; out float32 [rows, heads * vdim].
LLMK_API int llmk_mlstm_scan(float* out, long long out_stride, const float* proj, const float* partials, int splits,
                             long long split_stride, long long proj_stride, long long gate_col, const float* i_bias,
                             const float* f_bias, float cap, float q_scale, float* state, long long slot_stride, long long n_off,
                             long long m_off, const int* state_slots, const int* cu_tokens, int n_entries, int heads, int dim, int vdim,
                             int single, cudaStream_t stream) {
  if (n_entries == 0) return 0;
  LLMK_REQUIRE((proj != nullptr) != (partials != nullptr), "mlstm_scan: give proj or partials");
  LLMK_REQUIRE(dim > 0 && vdim > 0 && heads > 0 && cap > 0.f, "mlstm_scan: bad sizes or gate cap");
  LLMK_REQUIRE(n_entries <= 65535 && heads <= 65535, "mlstm_scan: too many entries or heads for one launch");
  LLMK_REQUIRE(n_off >= (long long)heads * dim * vdim && m_off >= n_off + (long long)heads * ((vdim + COLS - 1) / COLS) * dim,
               "mlstm_scan: the parts of a state row overlap");
  const Gates gt = {i_bias, f_bias, cap, q_scale};
  const State st = {state, slot_stride, n_off, m_off, state_slots};
  const dim3 grid((vdim + COLS - 1) / COLS, heads, n_entries);
  if (single) {
    LLMK_REQUIRE(dim <= DEC_MAX_DIM && vdim % 4 == 0, "mlstm_decode: key size %d (1 to %d) or value size %d (a multiple of 4)", dim,
                 DEC_MAX_DIM, vdim);
    LLMK_REQUIRE(slot_stride % 4 == 0 && (uintptr_t)state % 16 == 0, "mlstm_decode: the state must lie on the 16-byte grid");
    const MaybePartial<float> p{proj, partials, splits, split_stride};
    const bool vec = dim % 4 == 0 && proj_stride % 4 == 0 && p.vector_ok();
    launch_kernel(vec ? mlstm_decode_kernel<true> : mlstm_decode_kernel<false>, grid, dim3(DEC_THREADS), 0, stream, out, out_stride, p,
                  proj_stride, gate_col, gt, st, heads, dim, vdim);
    LLMK_LAUNCH_CHECK("mlstm_decode");
  }
  LLMK_REQUIRE(proj != nullptr, "mlstm_scan: partial results are for single tokens");
  LLMK_REQUIRE(dim <= ROWS * MAX_GROUPS, "mlstm_scan: key size %d (1 to %d)", dim, ROWS * MAX_GROUPS);
  const int groups = (dim + ROWS - 1) / ROWS;
  const size_t smem = ((size_t)2 * SC * groups * ROWS + SC * COLS + (size_t)SC * groups * COLS + SC * groups + 3 * SC) * sizeof(float);
  if (smem > 48 * 1024) cudaFuncSetAttribute(mlstm_scan_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  launch_kernel(mlstm_scan_kernel, grid, dim3(TX, groups), smem, stream, out, out_stride, proj, proj_stride, gate_col, gt, st, cu_tokens,
                heads, dim, vdim);
  LLMK_LAUNCH_CHECK("mlstm_scan");
}

// Entries of any length, chunk by chunk: q, k, v bfloat16 with one row stride (head h at column h * dim, of v h * vdim), z float32
// [n_tokens, >= 2 heads] the gates' pre-activations [i | f].  dim a multiple of 16 up to 256, vdim of 8.  E, e, fm: float32
// scratch of dim * vdim, dim and 4 floats per chunk and head for n_tokens / 64 + n_entries chunks.
LLMK_API int llmk_mlstm_chunks(float* out, long long out_stride, const void* q, const void* k, const void* v, long long stride,
                               const float* z, long long z_stride, const float* i_bias, const float* f_bias, float cap, float q_scale,
                               float* state, long long slot_stride, long long n_off, long long m_off, const int* state_slots,
                               const int* cu_tokens, int n_entries, int n_tokens, int heads, int dim, int vdim, float* E, float* e,
                               float* fm, cudaStream_t stream) {
  if (n_entries == 0 || n_tokens == 0) return 0;
  LLMK_REQUIRE(dim > 0 && dim % 16 == 0 && dim <= 256 && vdim > 0 && vdim % 8 == 0 && cap > 0.f,
               "mlstm_chunks: key size %d (a multiple of 16 up to 256) or value size %d (a multiple of 8)", dim, vdim);
  LLMK_REQUIRE(stride % 8 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)k % 16 == 0 && (uintptr_t)v % 16 == 0 && out_stride % 2 == 0 &&
                   (uintptr_t)out % 8 == 0 && slot_stride % 4 == 0 && n_off % 4 == 0 && (uintptr_t)state % 16 == 0 &&
                   (uintptr_t)E % 16 == 0 && (uintptr_t)e % 16 == 0 && (uintptr_t)fm % 16 == 0,
               "mlstm_chunks: operands off the 16-byte grid");
  LLMK_REQUIRE(n_entries <= 65535 && heads <= 65535, "mlstm_chunks: too many entries or heads for one launch");
  const Gates gt = {i_bias, f_bias, cap, q_scale};
  const State st = {state, slot_stride, n_off, m_off, state_slots};
  const Scratch sc = {E, e, fm};
  const int chunks = n_tokens / CC + n_entries, tiles = (vdim + VT - 1) / VT;
  const size_t smem1 = ((size_t)CC * (dim + PAD) + 3 * CC * VP) * sizeof(bf16);
  const size_t smem3 = ((size_t)2 * CC * (dim + PAD) + CC * VP + (size_t)3 * dim * VP) * sizeof(bf16);
  cudaFuncSetAttribute(mlstm_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
  auto outputs = dim == 128 ? mlstm_chunk_out_kernel<8> : dim == 64 ? mlstm_chunk_out_kernel<4>
               : dim == 32 ? mlstm_chunk_out_kernel<2> : mlstm_chunk_out_kernel<0>;
  cudaFuncSetAttribute(outputs, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3);
  launch_kernel(mlstm_chunk_state_kernel, dim3(chunks, heads, tiles), dim3(THREADS), smem1, stream, (const bf16*)k, (const bf16*)v, stride, z,
                z_stride, gt, cu_tokens, n_entries, heads, dim, vdim, sc);
  const size_t pairs = (size_t)heads * dim * vdim / 2 + (size_t)heads * dim / 2;
  launch_kernel(mlstm_chunk_chain_kernel, dim3((unsigned)((pairs + 255) / 256), n_entries), dim3(256), 0, stream, sc, st, cu_tokens, heads,
                dim, vdim, tiles);
  launch_kernel(outputs, dim3(chunks, heads, tiles), dim3(THREADS), smem3, stream, out, out_stride, (const bf16*)q, (const bf16*)k,
                (const bf16*)v, stride, z, z_stride, gt, st, cu_tokens, n_entries, heads, dim, vdim, sc);
  LLMK_LAUNCH_CHECK("mlstm_chunks");
}
