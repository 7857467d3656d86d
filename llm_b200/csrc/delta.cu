// The gated delta rule: a recurrent mixer whose matrix state per head is decayed, corrected toward the new value along the
// new key, and read out, token by token:
//
//   S <- g_t S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t         S [dim, vdim] per head
//   q_t, k_t unit vectors per head (x / sqrt(sum(x^2) + 1e-6)), q_t also times q_scale;
//   beta_t = sigmoid(b_t),  g_t = exp(-exp(A_log) softplus(a_t + dt_bias))                   one number per head and token
//
// or, with a decay per key channel (CH), g_t = diag(exp(-exp(A_log) softplus(z_t + dt_bias))), z_t and dt_bias [dim] per head: the
// rows of S decay each on its own, S^T k is taken over k times the decays, and everything else stays.
//
// Head h reads q/k head h / (heads / qk_heads).  The state is float32 and lives in the request's state slot (zero at
// admission); it is read at the start of an entry's tokens and written back at their end, so a whole prompt, a portion and a
// single token run the same arithmetic, in the same order, whatever else is in the batch.  Norms, beta, the decay, the
// state and every sum are float32; q, k, v, a, b are read in the projections' kind.
//
// The columns of S never mix: S^T k, the update and S^T q are all per column, and the read-out is taken from the decayed
// state before the write, o = g S^T q + u (k . q), so that both sums over the rows run side by side.  A warp owns eight
// columns of one head: its lanes are 8 row lanes x 4 column lanes, a lane keeps R consecutive rows of two columns in
// registers (R = a head's rows / 8, rounded up to 4, 8, 16 or 32), so a sum over the rows is R multiply-adds in a lane and
// three exchanges between the eight row lanes.  A CTA is WARPS warps (32 columns); its tokens are staged CHUNK at a time:
// the warps norm q and k into shared memory (a row lane's rows lie R + 4 floats apart there, which keeps the eight lanes'
// 16-byte loads on different banks), then every warp walks the chunk on its own, with the next chunk's loads already in
// flight.  (Two-wide float32 multiply-adds on a lane's two columns were tried: fewer instructions, but 927 us against 733 us
// for 2,048 tokens of 8 heads of 128 x 128: the walk is bound by the latency of its dependent steps, not by issue slots.)  The transition of a token is not
// diagonal, so a prompt is not cut into segments here: an entry's tokens run one after another in every CTA of its heads.
#include "common.cuh"

namespace {

#ifndef DELTA_UNROLL
#define DELTA_UNROLL 1
#endif
constexpr int WALK_UNROLL = DELTA_UNROLL;      // tokens of the walk that the compiler may interleave
constexpr int COLS = 2, ROW_LANES = 8, COL_LANES = 4, WARPS = 4, CHUNK = 16, VT = COLS * COL_LANES * WARPS;

__device__ __forceinline__ float softplus_d(float x) { return x > 20.f ? x : log1pf(expf(x)); }

struct DeltaArgs {
  float* out; long long out_stride;                       // [T, heads * vdim] float32
  const void *q, *k; long long qk_stride;                 // [T, qk_heads * dim]
  const void* v; long long v_stride;                      // [T, heads * vdim]
  const void *b, *a; long long b_stride, a_stride;        // b [T, heads]; a [T, heads], or (CH) float32 [T, heads * dim]
  const float *a_log, *dt_bias;                           // [heads]; (CH) dt_bias [heads * dim]
  float* state; long long slot_stride;                    // slot s at state + s * slot_stride: [heads, dim, vdim]
  const int *state_slots, *cu_tokens;
  int heads, qk_heads, dim, vdim;
  float q_scale, norm_eps;
};

template <typename T, int R, bool CH>
__global__ void __launch_bounds__(WARPS * 32)
delta_scan_kernel(DeltaArgs a) {
  extern __shared__ __align__(16) float smem[];
  pdl_launch_dependents();
  pdl_wait();
  constexpr int PITCH = R + 4, DP = ROW_LANES * PITCH;      // floats of one token's q (or k) in shared memory
  constexpr int PER = (ROW_LANES * R + 31) / 32;            // channels a lane stages of a token
  float* q_s = smem;                       // [CHUNK][DP]
  float* k_s = q_s + CHUNK * DP;           // [CHUNK][DP]
  float* v_s = k_s + CHUNK * DP;           // [CHUNK][VT]
  float* o_s = v_s + CHUNK * VT;           // [CHUNK][VT]
  float* g_s = o_s + CHUNK * VT;           // [CHUNK] decay, [CHUNK] beta, [CHUNK] k . q
  float* beta_s = g_s + CHUNK;
  float* kq_s = beta_s + CHUNK;
  float* kd_s = kq_s + CHUNK;              // CH: [CHUNK][DP] the keys as they are (k_s and q_s then hold them times the decays)
  float* gd_s = kd_s + CHUNK * DP;         // CH: [CHUNK][DP] the decays
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, tid = threadIdx.x;
  const int rl = lane & (ROW_LANES - 1), cl = lane >> 3;
  const int entry = blockIdx.z, head = blockIdx.y;
  const int qk_head = head / (a.heads / a.qk_heads);
  const int dim = a.dim, vdim = a.vdim;
  const int wcol = warp * (COLS * COL_LANES) + cl * COLS;       // the lane's first column within the CTA's VT
  const int col0 = blockIdx.x * VT + wcol;
  const int t0 = a.cu_tokens[entry], t1 = a.cu_tokens[entry + 1];
  if (t0 >= t1) return;
  using A = typename std::conditional<CH, float, T>::type;
  const T *q = (const T*)a.q, *k = (const T*)a.k, *v = (const T*)a.v, *pb = (const T*)a.b;
  const A* pa = (const A*)a.a;
  float* S_g = a.state + (size_t)a.state_slots[entry] * a.slot_stride + ((size_t)head * dim) * vdim;
  const float neg_a = -expf(a.a_log[head]), dt_b = CH ? 0.f : a.dt_bias[head];
  float dt_c[CH ? PER : 1];                // CH: the bias of the channels that this lane stages
  if (CH)
#pragma unroll
    for (int i = 0; i < PER; ++i) dt_c[CH ? i : 0] = lane + 32 * i < dim ? a.dt_bias[(size_t)head * dim + lane + 32 * i] : 0.f;

  float S[R][COLS];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int d = rl * R + i;
#pragma unroll
    for (int c = 0; c < COLS; ++c) S[i][c] = (d < dim && col0 + c < vdim) ? S_g[(size_t)d * vdim + col0 + c] : 0.f;
  }

  // What a thread brings of a chunk, requested one chunk ahead so that the loads land under the previous chunk's walk:
  // its warp's tokens (warp, warp + WARPS, ...) of q and k, PER channels a lane; lane j's b and a of the warp's j-th token;
  // and its share of the chunk's values.
  constexpr int TOK = CHUNK / WARPS, VREGS = CHUNK * VT / (WARPS * 32);
  T q_r[TOK][PER], k_r[TOK][PER], v_r[VREGS], b_r = T();
  A a_r = A(), z_r[CH ? TOK : 1][CH ? PER : 1];
  auto fetch = [&](int c0) {
    const int n = min(CHUNK, t1 - c0);
#pragma unroll
    for (int j = 0; j < TOK; ++j) {
      const int c = warp + j * WARPS;
      const size_t at = (size_t)(c0 + c) * a.qk_stride + (size_t)qk_head * dim;
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int d = lane + 32 * i;
        if (c < n && d < dim) {
          q_r[j][i] = q[at + d]; k_r[j][i] = k[at + d];
          if (CH) z_r[CH ? j : 0][CH ? i : 0] = pa[(size_t)(c0 + c) * a.a_stride + (size_t)head * dim + d];
        }
      }
    }
    if (lane < TOK && warp + lane * WARPS < n) {
      const size_t t = (size_t)(c0 + warp + lane * WARPS);
      b_r = pb[t * a.b_stride + head];
      if (!CH) a_r = pa[t * a.a_stride + head];
    }
#pragma unroll
    for (int i = 0; i < VREGS; ++i) {
      const int idx = tid + i * WARPS * 32, cc = blockIdx.x * VT + idx % VT;
      if (idx < n * VT && cc < vdim) v_r[i] = v[(size_t)(c0 + idx / VT) * a.v_stride + (size_t)head * vdim + cc];
    }
  };
  fetch(t0);

  for (int c0 = t0; c0 < t1; c0 += CHUNK) {
    const int n = min(CHUNK, t1 - c0);
    __syncthreads();                         // the previous chunk's outputs have been written out
    // unit q and k of this chunk's tokens, their product, the decay and beta: a warp norms its tokens side by side (the
    // sums of squares and the raw product of all of them go through one round of exchanges)
    {
      float qv[TOK][PER], kv[TOK][PER], red[TOK][3];
#pragma unroll
      for (int j = 0; j < TOK; ++j) {
        const bool live = warp + j * WARPS < n;
        red[j][0] = red[j][1] = red[j][2] = 0.f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
          const bool on = live && lane + 32 * i < dim;
          qv[j][i] = on ? to_f32(q_r[j][i]) : 0.f;
          kv[j][i] = on ? to_f32(k_r[j][i]) : 0.f;
          red[j][0] = fmaf(qv[j][i], qv[j][i], red[j][0]);
          red[j][1] = fmaf(kv[j][i], kv[j][i], red[j][1]);
          red[j][2] = fmaf(qv[j][i], kv[j][i], red[j][2]);
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int j = 0; j < TOK; ++j)
#pragma unroll
          for (int x = 0; x < 3; ++x) red[j][x] += __shfl_xor_sync(0xffffffffu, red[j][x], o);
#pragma unroll
      for (int j = 0; j < TOK; ++j) {
        const int c = warp + j * WARPS;
        if (c >= n) continue;
        const float rq = a.q_scale / sqrtf(red[j][0] + a.norm_eps), rk = 1.f / sqrtf(red[j][1] + a.norm_eps);
#pragma unroll
        for (int i = 0; i < PER; ++i) {
          const int d = lane + 32 * i;
          if (d < ROW_LANES * R) {
            const int at = c * DP + (d / R) * PITCH + d % R;
            float g = 1.f;
            if (CH) {
              g = d < dim ? expf(neg_a * softplus_d(to_f32(z_r[CH ? j : 0][CH ? i : 0]) + dt_c[CH ? i : 0])) : 0.f;
              kd_s[at] = kv[j][i] * rk;
              gd_s[at] = g;
            }
            q_s[at] = qv[j][i] * rq * g;
            k_s[at] = kv[j][i] * rk * g;
          }
        }
        if (lane == j) {
          kq_s[c] = red[j][2] * rq * rk;
          beta_s[c] = 1.f / (1.f + expf(-to_f32(b_r)));
          if (!CH) g_s[c] = expf(neg_a * softplus_d(to_f32(a_r) + dt_b));
        }
      }
    }
#pragma unroll
    for (int i = 0; i < VREGS; ++i) {
      const int idx = tid + i * WARPS * 32;
      if (idx < n * VT) v_s[idx] = blockIdx.x * VT + idx % VT < vdim ? to_f32(v_r[i]) : 0.f;
    }
    __syncthreads();
    if (c0 + CHUNK < t1) fetch(c0 + CHUNK);
#pragma unroll WALK_UNROLL
    for (int c = 0; c < n; ++c) {
      const float g = CH ? 1.f : g_s[c], beta = beta_s[c], kq = kq_s[c];      // CH: the decays are in k_s and q_s
      float kd[R];
      float pk[COLS][2], pq[COLS][2];          // two partial sums each: the chains of multiply-adds are half as long
#pragma unroll
      for (int cc = 0; cc < COLS; ++cc) pk[cc][0] = pk[cc][1] = pq[cc][0] = pq[cc][1] = 0.f;
#pragma unroll
      for (int i = 0; i < R; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(k_s + c * DP + rl * PITCH + i);
        const float4 q4 = *reinterpret_cast<const float4*>(q_s + c * DP + rl * PITCH + i);
        kd[i] = k4.x; kd[i + 1] = k4.y; kd[i + 2] = k4.z; kd[i + 3] = k4.w;
        const float qd[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int cc = 0; cc < COLS; ++cc) {
            pk[cc][j & 1] = fmaf(S[i + j][cc], kd[i + j], pk[cc][j & 1]);
            pq[cc][j & 1] = fmaf(S[i + j][cc], qd[j], pq[cc][j & 1]);
          }
      }
      float sk[COLS], sq[COLS];
#pragma unroll
      for (int cc = 0; cc < COLS; ++cc) { sk[cc] = pk[cc][0] + pk[cc][1]; sq[cc] = pq[cc][0] + pq[cc][1]; }
#pragma unroll
      for (int o = ROW_LANES / 2; o > 0; o >>= 1) {
#pragma unroll
        for (int cc = 0; cc < COLS; ++cc) {
          sk[cc] += __shfl_xor_sync(0xffffffffu, sk[cc], o);
          sq[cc] += __shfl_xor_sync(0xffffffffu, sq[cc], o);
        }
      }
      const float2 v2 = *reinterpret_cast<const float2*>(v_s + c * VT + wcol);
      const float vv[COLS] = {v2.x, v2.y};
      float u[COLS], o2[COLS];
#pragma unroll
      for (int cc = 0; cc < COLS; ++cc) {
        u[cc] = beta * (vv[cc] - g * sk[cc]);
        o2[cc] = fmaf(u[cc], kq, g * sq[cc]);
      }
      if (CH) {
#pragma unroll
        for (int i = 0; i < R; i += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(kd_s + c * DP + rl * PITCH + i);
          const float4 g4 = *reinterpret_cast<const float4*>(gd_s + c * DP + rl * PITCH + i);
          const float kr[4] = {k4.x, k4.y, k4.z, k4.w}, gr[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
          for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int cc = 0; cc < COLS; ++cc) S[i + j][cc] = fmaf(kr[j], u[cc], gr[j] * S[i + j][cc]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < R; ++i)
#pragma unroll
          for (int cc = 0; cc < COLS; ++cc) S[i][cc] = fmaf(kd[i], u[cc], g * S[i][cc]);
      }
      if (rl == 0) *reinterpret_cast<float2*>(o_s + c * VT + wcol) = make_float2(o2[0], o2[1]);
    }
    __syncthreads();
    for (int idx = tid; idx < n * VT; idx += WARPS * 32) {
      const int c = idx / VT, cc = blockIdx.x * VT + idx % VT;
      if (cc < vdim) a.out[(size_t)(c0 + c) * a.out_stride + (size_t)head * vdim + cc] = o_s[idx];
    }
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int d = rl * R + i;
    if (d >= dim) continue;
#pragma unroll
    for (int c = 0; c < COLS; ++c)
      if (col0 + c < vdim) S_g[(size_t)d * vdim + col0 + c] = S[i][c];
  }
}

template <typename T, int R, bool CH>
int launch_delta(const DeltaArgs& a, int n_entries, cudaStream_t stream) {
  const size_t smem = ((size_t)(CH ? 4 : 2) * CHUNK * ROW_LANES * (R + 4) + 2 * CHUNK * VT + 3 * CHUNK) * sizeof(float);
  if (smem > 48 * 1024) cudaFuncSetAttribute(delta_scan_kernel<T, R, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  const dim3 grid((a.vdim + VT - 1) / VT, a.heads, n_entries);
  launch_kernel(delta_scan_kernel<T, R, CH>, grid, dim3(WARPS * 32), smem, stream, a);
  LLMK_LAUNCH_CHECK("delta_scan");
}

template <typename T, bool CH>
int launch_delta_of(const DeltaArgs& a, int n_entries, cudaStream_t stream) {
  if (a.dim <= 32) return launch_delta<T, 4, CH>(a, n_entries, stream);
  if (a.dim <= 64) return launch_delta<T, 8, CH>(a, n_entries, stream);
  if (a.dim <= 128) return launch_delta<T, 16, CH>(a, n_entries, stream);
  return launch_delta<T, 32, CH>(a, n_entries, stream);
}

// ---- prompts: the rule chunk by chunk ---------------------------------------------------------------------------
// Within a chunk of CC tokens the rule is linear in the state S_0 that enters the chunk.  With L_t the running sum of
// log g over the chunk's tokens (so that exp(L_t - L_s) is the decay from token s to token t):
//     u_t = beta_t (v_t - exp(L_t) S_0^T k_t - sum_{s<t} exp(L_t - L_s) (k_t . k_s) u_s)
// is a unit lower triangular system (I + A) U = beta V - (beta exp(L) K) S_0 with A_ts = beta_t exp(L_t - L_s) (k_t . k_s), so
//     U = W - Y S_0,   W = (I + A)^-1 (beta V),   Y = (I + A)^-1 (beta exp(L) K)
//     o_t = (exp(L_t) q_t)^T S_0 + sum_{s<=t} B_ts u_s,   B_ts = exp(L_t - L_s) (q_t . k_s)
//     S_C = exp(L_C) S_0 + sum_s (exp(L_C - L_s) k_s) u_s^T
// W, Y, B and the scaled q and k do not depend on the state: delta_prepare makes them for every chunk of the step side by
// side (a CTA per chunk and head: unit norms, the two Gram matrices, forward substitution with a column per thread) and
// leaves them chunk by chunk, padded with zeros to whole chunks, Y and the scaled q with the tokens innermost.
// delta_chunk_walk then runs an entry's chunks one after another and does only what the chain needs: U = W - Y S_0 (left in
// W's place) and the next S_0 (left for every chunk), two small matrix products on the CUDA cores with the operands in
// shared memory (asynchronous copies, the next chunk's under this chunk's arithmetic), the first with its sum over the state's
// rows split over the warps, the state's tile in registers from chunk to chunk and mirrored in shared memory.
// delta_chunk_out makes the outputs of all chunks side by side again.  What is left of the chain from token to token is one
// step per chunk.  All of it float32; the sums of a token are grouped by where its chunk begins, which moves results by
// rounding only.
//
// With a decay per key channel (CH) L_t is a vector over the channels and the decays stand inside the Gram matrices,
//     A_ts = beta_t sum_d exp(L_td - L_sd) k_td k_sd,    B_ts alike with q_t,
// while Y, the scaled q and k and the end decay take them channel by channel and the walk stays as it is.  exp(L_t) and
// exp(-L_s) cannot be taken apart (the second overflows), but within reach of a token r between s and t both exp(L_t - L_r) and
// exp(L_r - L_s) are at most one: the chunk is cut into blocks of CB tokens, the Gram entries of two different blocks are
// plain products of rows scaled to the last token before the later block, and only those within a block take an exponential
// for every channel and pair.
constexpr int CC = 32, CB = 8;

struct PrepArgs {
  const void *q, *k; long long qk_stride;
  const void* v; long long v_stride;
  const void *b, *a; long long b_stride, a_stride;
  const float *a_log, *dt_bias;
  const int* cu_tokens; int n_entries;
  int heads, qk_heads, dim, vdim;
  float q_scale, norm_eps;
  // per chunk c and head h, at (c * heads + h) * size: YQ [dim][2 CC] (Y's tokens, then the scaled q's), K [CC][dim],
  // W [CC][vdim], B [CC][CC], G [1] (the chunk's whole decay; CH: [dim])
  float *YQ, *K, *W, *B, *G;
  bool vec;                 // q, k and (CH) a and dt_bias may be read four channels at a time
};

// The chunk with the running number idx: its first token and its length, or false when the step has fewer chunks.
__device__ __forceinline__ bool chunk_of(const int* cu_tokens, int n_entries, int idx, int& c0, int& n) {
  for (int e = 0; e < n_entries; ++e) {
    const int t0 = cu_tokens[e], len = cu_tokens[e + 1] - t0, chunks = (len + CC - 1) / CC;
    if (idx < chunks) { c0 = t0 + idx * CC; n = min(CC, len - idx * CC); return true; }
    idx -= chunks;
  }
  return false;
}

constexpr int PT = 256;                      // threads of a preparing CTA
constexpr int FAR_S = CB * (CC / CB) * (CC / CB - 1) / 2;      // rows of keys scaled to the token before a later block, over all blocks
constexpr float LOG2_E = 1.44269504088896340736f;

// Floats of shared memory: unit k and q [CC][pitch], A with its rows innermost [CC][CC + 4], beta [CC], the decays' running sums
// ([CC], CH: [CC][pitch]) and (CH) the scaled rows: k before each block [FAR_S][pitch], k and q of the blocks [2][CC - CB][pitch].
__host__ __device__ inline int prepare_pitch(int dim) { return (dim + 3) / 4 * 4 + 4; }
inline size_t prepare_floats(int dim, bool ch) {
  const int p = prepare_pitch(dim);
  return (size_t)2 * CC * p + CC * (CC + 4) + CC + (ch ? (size_t)(CC + FAR_S + 2 * (CC - CB)) * p : (size_t)CC);
}

template <typename T, bool CH>
__global__ void __launch_bounds__(PT, 2)
delta_prepare_kernel(PrepArgs a) {
  extern __shared__ __align__(16) float smem[];
  pdl_launch_dependents();
  pdl_wait();
  int c0, n;
  if (!chunk_of(a.cu_tokens, a.n_entries, blockIdx.x, c0, n)) return;
  const int head = blockIdx.y, qk_head = head / (a.heads / a.qk_heads);
  const int dim = a.dim, vdim = a.vdim, pitch = prepare_pitch(dim), dim4 = pitch - 4;
  const size_t unit = (size_t)blockIdx.x * a.heads + head;
  constexpr int AP = CC + 4;
  float* kn = smem;                        // [CC][pitch], zeros behind dim
  float* qn = kn + CC * pitch;
  float* At = qn + CC * pitch;             // [CC][AP]: At[s][t] = A_ts, zero unless s < t
  float* beta_s = At + CC * AP;
  float* L_s = beta_s + CC;                // the running sums of log2 g
  float* kr_s = L_s + CC * pitch;          // CH
  float* xr_s = kr_s + FAR_S * pitch;      // CH
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const T *q = (const T*)a.q, *k = (const T*)a.k, *v = (const T*)a.v, *pb = (const T*)a.b;
  using A = typename std::conditional<CH, float, T>::type;
  const A* pa = (const A*)a.a;
  const float neg_a = -expf(a.a_log[head]) * LOG2_E, dt_b = CH ? 0.f : a.dt_bias[head];

  // q, k and the logarithms of the decays as they come; beta.  Every loop over channels takes four of them a thread; loads go
  // to clamped places, so that none waits for a test.
  const int quads = dim4 / 4;
  auto put4 = [](float* p, float x, float y, float z, float w) { *reinterpret_cast<float4*>(p) = make_float4(x, y, z, w); };
  auto at4 = [](const float* p) { return *reinterpret_cast<const float4*>(p); };
#pragma unroll 4
  for (int i = tid; i < CC * quads; i += PT) {
    const int t = i / quads, d = 4 * (i % quads);
    const size_t row = (size_t)(c0 + min(t, n - 1));
    const T *qp = q + row * a.qk_stride + (size_t)qk_head * dim, *kp = k + row * a.qk_stride + (size_t)qk_head * dim;
    float qv[4], kv[4], zv[4] = {0.f, 0.f, 0.f, 0.f}, bv[4] = {0.f, 0.f, 0.f, 0.f};
    if (a.vec) {
      Vec4<T>::load(qp + d, qv); Vec4<T>::load(kp + d, kv);
      if constexpr (CH) { Vec4<float>::load(pa + row * a.a_stride + (size_t)head * dim + d, zv); Vec4<float>::load(a.dt_bias + (size_t)head * dim + d, bv); }
    } else {
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int e = min(d + x, dim - 1);
        qv[x] = to_f32(qp[e]); kv[x] = to_f32(kp[e]);
        if (CH) { zv[x] = to_f32(pa[row * a.a_stride + (size_t)head * dim + e]); bv[x] = a.dt_bias[(size_t)head * dim + e]; }
      }
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const bool on = t < n && d + x < dim;
      qv[x] = on ? qv[x] : 0.f; kv[x] = on ? kv[x] : 0.f;
      if (CH) zv[x] = on ? neg_a * softplus_d(zv[x] + bv[x]) : 0.f;
    }
    put4(qn + t * pitch + d, qv[0], qv[1], qv[2], qv[3]);
    put4(kn + t * pitch + d, kv[0], kv[1], kv[2], kv[3]);
    if (CH) put4(L_s + t * pitch + d, zv[0], zv[1], zv[2], zv[3]);
  }
  if (tid < CC) {
    const int t = tid;
    beta_s[t] = t < n ? 1.f / (1.f + expf(-to_f32(pb[(size_t)(c0 + t) * a.b_stride + head]))) : 0.f;
    if (!CH) L_s[t] = t < n ? neg_a * softplus_d(to_f32(pa[(size_t)(c0 + t) * a.a_stride + head]) + dt_b) : 0.f;
  }
  for (int i = tid; i < CC * AP; i += PT) At[i] = 0.f;
  for (int i = tid; i < CC * CC; i += PT)
    if (i % CC > i / CC) a.B[unit * CC * CC + i] = 0.f;
  __syncthreads();
  // unit q and k: a warp per token; the running sums
  for (int t = warp; t < CC; t += PT / 32) {
    float sq = 0.f, sk = 0.f;
    for (int d = lane; d < dim; d += 32) {
      sq = fmaf(qn[t * pitch + d], qn[t * pitch + d], sq);
      sk = fmaf(kn[t * pitch + d], kn[t * pitch + d], sk);
    }
    const float rq = a.q_scale / sqrtf(warp_sum(sq) + a.norm_eps), rk = 1.f / sqrtf(warp_sum(sk) + a.norm_eps);
    for (int d = lane; d < dim; d += 32) { qn[t * pitch + d] *= rq; kn[t * pitch + d] *= rk; }
  }
  if (CH) {
    for (int d = tid; d < dim; d += PT) {
      float run = 0.f;
#pragma unroll
      for (int t = 0; t < CC; ++t) { run += L_s[t * pitch + d]; L_s[t * pitch + d] = run; }
    }
  } else if (tid == 0) {
    float run = 0.f;
#pragma unroll
    for (int t = 0; t < CC; ++t) { run += L_s[t]; L_s[t] = run; }
  }
  __syncthreads();
  // the two Gram matrices with their decays
  auto dot4 = [](const float4& x, const float4& y, float s) { return fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, s)))); };
  if (CH) {
    // rows scaled to and from the token before each block but the first
    auto scaled = [&](const float4& x, const float4& hi, const float4& lo) {
      return make_float4(x.x * exp2f(hi.x - lo.x), x.y * exp2f(hi.y - lo.y), x.z * exp2f(hi.z - lo.z), x.w * exp2f(hi.w - lo.w));
    };
#pragma unroll 2
    for (int i = tid; i < FAR_S * quads; i += PT) {
      int s2 = i / quads, blk = 1;
      const int d = 4 * (i % quads), row = s2;
      while (s2 >= blk * CB) { s2 -= blk * CB; ++blk; }
      *reinterpret_cast<float4*>(kr_s + row * pitch + d) = scaled(at4(kn + s2 * pitch + d), at4(L_s + (blk * CB - 1) * pitch + d), at4(L_s + s2 * pitch + d));
    }
#pragma unroll 2
    for (int i = tid; i < 2 * (CC - CB) * quads; i += PT) {
      const int row = i / quads, d = 4 * (i % quads), t = row % (CC - CB) + CB;
      *reinterpret_cast<float4*>(xr_s + row * pitch + d) =
          scaled(at4((row < CC - CB ? kn : qn) + t * pitch + d), at4(L_s + t * pitch + d), at4(L_s + (t / CB * CB - 1) * pitch + d));
    }
    // pairs within a block: four threads a pair, an exponential for every channel
    constexpr int PAIRS = CB * (CB + 1) / 2;
    static_assert(CC / CB * PAIRS % 8 == 0, "a warp's eight pairs are all there or none");
    for (int w = tid / 4; w < CC / CB * PAIRS; w += PT / 4) {
      const int blk = w / PAIRS;
      int i = 0, left = w % PAIRS;
      while (left > i) { left -= i + 1; ++i; }                // the pair (i, left), left <= i, of the block's lower triangle
      const int t = blk * CB + i, s2 = blk * CB + left;
      float kk = 0.f, qk = 0.f;
      for (int d = 4 * (tid % 4); d < dim4; d += 16) {
        const float4 lt = at4(L_s + t * pitch + d), ls = at4(L_s + s2 * pitch + d);
        float4 x = at4(kn + s2 * pitch + d);
        x.x *= exp2f(lt.x - ls.x); x.y *= exp2f(lt.y - ls.y); x.z *= exp2f(lt.z - ls.z); x.w *= exp2f(lt.w - ls.w);
        kk = dot4(at4(kn + t * pitch + d), x, kk);
        qk = dot4(at4(qn + t * pitch + d), x, qk);
      }
      kk += __shfl_xor_sync(0xffffffffu, kk, 1); kk += __shfl_xor_sync(0xffffffffu, kk, 2);
      qk += __shfl_xor_sync(0xffffffffu, qk, 1); qk += __shfl_xor_sync(0xffffffffu, qk, 2);
      if (tid % 4 == 0) {
        if (s2 < t) At[s2 * AP + t] = kk * beta_s[t];
        a.B[unit * CC * CC + t * CC + s2] = qk;
      }
    }
    __syncthreads();
    // pairs of two blocks: a thread a token and two earlier ones
    for (int w = tid; w < CB * FAR_S / 2; w += PT) {
      const int i = w % CB;
      int s2 = w / CB * 2, blk = 1;
      const int far = s2;
      while (s2 >= blk * CB) { s2 -= blk * CB; ++blk; }
      const int t = blk * CB + i;
      const float *xk = xr_s + (t - CB) * pitch, *xq = xk + (CC - CB) * pitch, *y0 = kr_s + far * pitch, *y1 = y0 + pitch;
      float kk0 = 0.f, kk1 = 0.f, qk0 = 0.f, qk1 = 0.f;
#pragma unroll 2
      for (int d = 0; d < dim4; d += 4) {
        const float4 k4 = at4(xk + d), q4 = at4(xq + d), u = at4(y0 + d), w4 = at4(y1 + d);
        kk0 = dot4(k4, u, kk0); kk1 = dot4(k4, w4, kk1);
        qk0 = dot4(q4, u, qk0); qk1 = dot4(q4, w4, qk1);
      }
      At[s2 * AP + t] = kk0 * beta_s[t]; At[(s2 + 1) * AP + t] = kk1 * beta_s[t];
      *reinterpret_cast<float2*>(a.B + unit * CC * CC + t * CC + s2) = make_float2(qk0, qk1);
    }
  } else {
    // a thread two tokens and two others
    static_assert(CC / 2 * (CC / 2) == PT, "a tile of 2 x 2 pairs a thread");
    const int t = 2 * (tid / (CC / 2)), s2 = 2 * (tid % (CC / 2));
    if (s2 <= t) {
      float kk[2][2] = {{0.f, 0.f}, {0.f, 0.f}}, qk[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
#pragma unroll 2
      for (int d = 0; d < dim4; d += 4) {
        const float4 x[2] = {at4(kn + s2 * pitch + d), at4(kn + (s2 + 1) * pitch + d)};
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const float4 k4 = at4(kn + (t + i) * pitch + d), q4 = at4(qn + (t + i) * pitch + d);
#pragma unroll
          for (int j = 0; j < 2; ++j) { kk[i][j] = dot4(k4, x[j], kk[i][j]); qk[i][j] = dot4(q4, x[j], qk[i][j]); }
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const float e = exp2f(L_s[t + i] - L_s[s2 + j]);
          if (s2 + j < t + i) At[(s2 + j) * AP + t + i] = kk[i][j] * e * beta_s[t + i];
          if (s2 + j <= t + i) a.B[unit * CC * CC + (t + i) * CC + s2 + j] = qk[i][j] * e;
        }
    }
  }
  __syncthreads();
  // forward substitution: a thread per column of [beta V | beta exp(L) K], the column in registers, earlier tokens taken off later
  // ones token by token
  for (int col = tid; col < vdim + dim; col += PT) {
    float x[CC];
    const bool is_v = col < vdim;
    const int d = col - vdim;
    if (is_v) {
      const T* vp = v + (size_t)c0 * a.v_stride + (size_t)head * vdim + col;
#pragma unroll
      for (int t = 0; t < CC; ++t) x[t] = to_f32(vp[(size_t)min(t, n - 1) * a.v_stride]);
#pragma unroll
      for (int t = 0; t < CC; ++t) x[t] *= beta_s[t];        // beta is zero behind the chunk's last token
    } else {
#pragma unroll
      for (int t = 0; t < CC; ++t) x[t] = beta_s[t] * exp2f(CH ? L_s[t * pitch + d] : L_s[t]) * kn[t * pitch + d];
    }
#pragma unroll
    for (int s2 = 0; s2 < CC - 1; ++s2) {
#pragma unroll
      for (int t = (s2 + 1) / 4 * 4; t < CC; t += 4) {
        const float4 f = at4(At + s2 * AP + t);               // zero up to token s2
        if (t > s2) x[t] = fmaf(-f.x, x[s2], x[t]);
        if (t + 1 > s2) x[t + 1] = fmaf(-f.y, x[s2], x[t + 1]);
        if (t + 2 > s2) x[t + 2] = fmaf(-f.z, x[s2], x[t + 2]);
        if (t + 3 > s2) x[t + 3] = fmaf(-f.w, x[s2], x[t + 3]);
      }
    }
    if (is_v) {
#pragma unroll
      for (int t = 0; t < CC; ++t) a.W[(unit * CC + t) * vdim + col] = x[t];
    } else {                                 // Y with the tokens innermost: the column as it lies in the registers
      float* dst = a.YQ + (unit * dim + d) * (2 * CC);
#pragma unroll
      for (int t = 0; t < CC; t += 4) *reinterpret_cast<float4*>(dst + t) = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
    }
  }
  // q and k with the decays that follow need: to the token from the chunk's start, from the token to the chunk's end
  for (int i = tid; i < dim * (CC / 4); i += PT) {
    const int d = i % dim, t = i / dim * 4;
    float y[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) y[x] = exp2f(CH ? L_s[(t + x) * pitch + d] : L_s[t + x]) * qn[(t + x) * pitch + d];
    *reinterpret_cast<float4*>(a.YQ + (unit * dim + d) * (2 * CC) + CC + t) = make_float4(y[0], y[1], y[2], y[3]);
  }
#pragma unroll 2
  for (int i = tid; i < CC * quads; i += PT) {
    const int t = i / quads, d = 4 * (i % quads);
    const float4 k4 = at4(kn + t * pitch + d);                // zero behind the last token
    float y[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
    for (int x = 0; x < 4; ++x) y[x] *= exp2f(CH ? L_s[(n - 1) * pitch + d + x] - L_s[t * pitch + d + x] : L_s[n - 1] - L_s[t]);
    float* dst = a.K + (unit * CC + t) * dim + d;
    if (dim % 4 == 0) put4(dst, y[0], y[1], y[2], y[3]);
    else
#pragma unroll
      for (int x = 0; x < 4; ++x)
        if (d + x < dim) dst[x] = y[x];
  }
  if (CH)
    for (int d = tid; d < dim; d += PT) a.G[unit * dim + d] = exp2f(L_s[(n - 1) * pitch + d]);
  else if (tid == 0)
    a.G[unit] = exp2f(L_s[n - 1]);
}

struct WalkArgs {
  const float *YQ, *K, *G;
  float *W, *S;             // W [CC][vdim] becomes U; S [dim][vdim]: the state that enters the chunk
  float* state; long long slot_stride;
  const int *state_slots, *cu_tokens;
  int heads, dim, vdim;
};

__device__ __forceinline__ void cp_async16(void* smem_dst, const void* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(smem_dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// DPAD: a head's rows rounded up to 32, 64, 128 or 256; WV: value columns a CTA owns (16, or 8 where there would be few CTAs).
constexpr int WT = 256;                      // threads of a walking CTA

template <int DPAD, int WV>
struct WalkShape {
  static constexpr int C = 2;                                         // columns of a thread in both products
  static constexpr int R1 = 4, SLICE = CC / R1 * (WV / C);            // Y S_0: rows of a thread, threads of a slice of the sum
  static constexpr int KS = WT / SLICE, DEPTH = DPAD / KS;            // slices, and the state's rows in each
  static constexpr int TX = WV / C, TY = WT / TX, R2 = DPAD / TY;     // K^T U: the threads as TY x TX, rows of a thread
  static constexpr int STAGE = DPAD * CC + CC * DPAD + CC * WV;       // floats of one stage: Y, K, W
  static constexpr size_t SMEM = (size_t)(2 * STAGE + DPAD * WV + KS * CC * WV + CC * WV) * sizeof(float);
  static_assert(R2 >= 1 && DEPTH >= 1 && KS * DEPTH == DPAD && R2 * TY == DPAD, "the products divide among the threads");
};

template <int DPAD, int WV, bool CH>
__global__ void __launch_bounds__(WT)
delta_chunk_walk_kernel(WalkArgs a) {
  using Sh = WalkShape<DPAD, WV>;
  constexpr int R1 = Sh::R1, R2 = Sh::R2;
  extern __shared__ __align__(16) float smem[];
  pdl_launch_dependents();
  pdl_wait();
  float* S_s = smem + 2 * Sh::STAGE;        // [DPAD][WV]: the state as the first product reads it
  float* part_s = S_s + DPAD * WV;          // [KS][CC][WV]
  float* u_s = part_s + Sh::KS * CC * WV;   // [CC][WV]
  const int tid = threadIdx.x, ty = tid / Sh::TX, tx = tid % Sh::TX;
  const int ks = tid / Sh::SLICE, ry = (tid % Sh::SLICE) / (WV / 2), cx = tid % (WV / 2);
  const int entry = blockIdx.z, head = blockIdx.y;
  const int dim = a.dim, vdim = a.vdim, colb = blockIdx.x * WV, col = colb + 2 * tx;
  const int t0 = a.cu_tokens[entry], t1 = a.cu_tokens[entry + 1];
  if (t0 >= t1) return;
  int chunk = 0;                            // the running number of the entry's first chunk
  for (int e = 0; e < entry; ++e) chunk += (a.cu_tokens[e + 1] - a.cu_tokens[e] + CC - 1) / CC;
  const bool vec = dim % 4 == 0 && vdim % 4 == 0, even = vdim % 2 == 0;
  float* S_g = a.state + (size_t)a.state_slots[entry] * a.slot_stride + ((size_t)head * dim) * vdim;
  float S[R2][2];                           // rows R2 ty .., columns 2 tx ..
  auto put = [&](float* dst) {              // the thread's tile of the state, to a [dim][vdim] array
    const bool pairs = even && (uintptr_t)dst % 8 == 0;
#pragma unroll
    for (int i = 0; i < R2; ++i) {
      const int d = ty * R2 + i;
      if (d >= dim) continue;
      float* at = dst + (size_t)d * vdim + col;
      if (pairs && col < vdim) *reinterpret_cast<float2*>(at) = make_float2(S[i][0], S[i][1]);
      else
#pragma unroll
        for (int c = 0; c < 2; ++c)
          if (col + c < vdim) at[c] = S[i][c];
    }
  };
#pragma unroll
  for (int i = 0; i < R2; ++i) {
    const int d = ty * R2 + i;
#pragma unroll
    for (int c = 0; c < 2; ++c) S[i][c] = (d < dim && col + c < vdim) ? S_g[(size_t)d * vdim + col + c] : 0.f;
    *reinterpret_cast<float2*>(S_s + d * WV + 2 * tx) = make_float2(S[i][0], S[i][1]);
  }
  // request the operands of chunk number c into a stage (they are padded with zeros to whole chunks where they were made)
  auto issue = [&](int c, float* st) {
    const size_t unit = (size_t)c * a.heads + head;
    float *y_s = st, *k_s = st + DPAD * CC, *w_s = k_s + CC * DPAD;
    const float *y = a.YQ + unit * dim * 2 * CC, *k = a.K + unit * CC * dim, *w = a.W + unit * CC * vdim;
    for (int i = tid; i < dim * CC / 4; i += WT) cp_async16(y_s + 4 * i, y + (size_t)(i / (CC / 4)) * 2 * CC + 4 * (i % (CC / 4)));
    if (vec) {
      if (dim == DPAD)
        for (int i = tid; i < CC * DPAD / 4; i += WT) cp_async16(k_s + 4 * i, k + 4 * i);
      else
        for (int i = tid; i < CC * dim / 4; i += WT) cp_async16(k_s + (4 * i) / dim * DPAD + (4 * i) % dim, k + 4 * i);
      for (int i = tid; i < CC * WV / 4; i += WT) {
        const int c4 = (4 * i) % WV;
        if (colb + c4 < vdim) cp_async16(w_s + 4 * i, w + (size_t)((4 * i) / WV) * vdim + colb + c4);
      }
    } else {
      for (int i = tid; i < CC * dim; i += WT) k_s[(i / dim) * DPAD + i % dim] = k[i];
      for (int i = tid; i < CC * WV; i += WT)
        if (colb + i % WV < vdim) w_s[i] = w[(size_t)(i / WV) * vdim + colb + i % WV];
    }
    cp_async_commit();
  };
  // rows of Y and K beyond the head's and columns of W beyond the values' are never copied: they stay zero
  for (int i = tid; i < 2 * Sh::STAGE; i += WT) smem[i] = 0.f;
  __syncthreads();
  issue(chunk, smem);
  int at_stage = 0;
  for (int c0 = t0; c0 < t1; c0 += CC, ++chunk, at_stage ^= 1) {
    const size_t unit = (size_t)chunk * a.heads + head;
    const float *y_s = smem + at_stage * Sh::STAGE, *k_s = y_s + DPAD * CC, *w_s = k_s + CC * DPAD;
    float g_end[CH ? R2 : 1];
    if (CH) {
#pragma unroll
      for (int i = 0; i < R2; ++i) g_end[CH ? i : 0] = ty * R2 + i < dim ? a.G[unit * dim + ty * R2 + i] : 0.f;
    } else {
      g_end[0] = a.G[unit];
    }
    put(a.S + unit * dim * vdim);            // under the waits below
    if (c0 + CC < t1) {
      issue(chunk + 1, smem + (at_stage ^ 1) * Sh::STAGE);      // that stage's last readers passed the barrier below
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();                         // the stage has landed; S_s holds the state that enters the chunk
    {                                        // this slice's share of Y S_0: rows R1 ry .., columns 2 cx ..
      float acc[R1][2];
#pragma unroll
      for (int i = 0; i < R1; ++i) acc[i][0] = acc[i][1] = 0.f;
#pragma unroll 8
      for (int x = 0; x < Sh::DEPTH; ++x) {
        const int d = ks * Sh::DEPTH + x;
        const float4 y4 = *reinterpret_cast<const float4*>(y_s + d * CC + R1 * ry);
        const float2 s2 = *reinterpret_cast<const float2*>(S_s + d * WV + 2 * cx);
        const float yv[R1] = {y4.x, y4.y, y4.z, y4.w};
#pragma unroll
        for (int i = 0; i < R1; ++i) {
          acc[i][0] = fmaf(yv[i], s2.x, acc[i][0]);
          acc[i][1] = fmaf(yv[i], s2.y, acc[i][1]);
        }
      }
#pragma unroll
      for (int i = 0; i < R1; ++i)
        *reinterpret_cast<float2*>(part_s + (ks * CC + R1 * ry + i) * WV + 2 * cx) = make_float2(acc[i][0], acc[i][1]);
    }
    __syncthreads();
#pragma unroll
    for (int i = tid; i < CC * WV; i += WT) {
      float u = w_s[i];
#pragma unroll
      for (int k = 0; k < Sh::KS; ++k) u -= part_s[k * CC * WV + i];
      u_s[i] = u;
      if (colb + i % WV < vdim) a.W[(unit * CC + i / WV) * vdim + colb + i % WV] = u;
    }
    __syncthreads();
    // the state at the chunk's end: decays times S_0, plus (scaled K)^T U
#pragma unroll
    for (int i = 0; i < R2; ++i) { S[i][0] *= g_end[CH ? i : 0]; S[i][1] *= g_end[CH ? i : 0]; }
#pragma unroll 8
    for (int s2 = 0; s2 < CC; ++s2) {
      const float2 u2 = *reinterpret_cast<const float2*>(u_s + s2 * WV + 2 * tx);
      const float* kr = k_s + s2 * DPAD + ty * R2;
      float kv[R2];
      if constexpr (R2 % 4 == 0) {
#pragma unroll
        for (int i = 0; i < R2; i += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(kr + i);
          kv[i] = k4.x; kv[i + 1] = k4.y; kv[i + 2] = k4.z; kv[i + 3] = k4.w;
        }
      } else if constexpr (R2 == 2) {
        const float2 k2 = *reinterpret_cast<const float2*>(kr);
        kv[0] = k2.x; kv[1] = k2.y;
      } else {
        kv[0] = kr[0];
      }
#pragma unroll
      for (int i = 0; i < R2; ++i) {
        S[i][0] = fmaf(kv[i], u2.x, S[i][0]);
        S[i][1] = fmaf(kv[i], u2.y, S[i][1]);
      }
    }
    // every reader of the old S_s passed the second barrier above
#pragma unroll
    for (int i = 0; i < R2; ++i) *reinterpret_cast<float2*>(S_s + (ty * R2 + i) * WV + 2 * tx) = make_float2(S[i][0], S[i][1]);
    __syncthreads();                         // this stage may be overwritten
  }
  put(S_g);
}

template <int DPAD, int WV, bool CH>
int launch_walk(const WalkArgs& a, int n_entries, cudaStream_t stream) {
  constexpr size_t smem = WalkShape<DPAD, WV>::SMEM;
  if (smem > 48 * 1024) cudaFuncSetAttribute(delta_chunk_walk_kernel<DPAD, WV, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  launch_kernel(delta_chunk_walk_kernel<DPAD, WV, CH>, dim3((a.vdim + WV - 1) / WV, a.heads, n_entries), dim3(WT), smem, stream, a);
  LLMK_LAUNCH_CHECK("delta_chunk_walk");
}

template <int DPAD, bool CH>
int launch_walk_of(const WalkArgs& a, int n_entries, cudaStream_t stream) {
  if (DPAD >= 64 && (long long)(a.vdim + 15) / 16 * a.heads * n_entries < llmk_sm_count())
    return launch_walk<DPAD, DPAD >= 64 ? 8 : 16, CH>(a, n_entries, stream);
  return launch_walk<DPAD, 16, CH>(a, n_entries, stream);
}

// The outputs of a chunk: o_t = (scaled q_t)^T S_0 + sum_{s <= t} B_ts u_s; a CTA makes OV columns of one head's chunk, a thread 4
// tokens x 4 columns.  Grid (chunks, heads, column tiles).
constexpr int OV = 64, OT = CC / 4 * (OV / 4), BP = CC + 4;

struct OutArgs {
  float* out; long long out_stride;
  const float *YQ, *B, *U, *S;
  const int* cu_tokens; int n_entries;
  int heads, dim, vdim;
};

__global__ void __launch_bounds__(OT)
delta_chunk_out_kernel(OutArgs a) {
  extern __shared__ __align__(16) float smem[];
  pdl_launch_dependents();
  pdl_wait();
  int c0, n;
  if (!chunk_of(a.cu_tokens, a.n_entries, blockIdx.x, c0, n)) return;
  const int head = blockIdx.y, colb = blockIdx.z * OV, dim = a.dim, vdim = a.vdim, tid = threadIdx.x;
  const size_t unit = (size_t)blockIdx.x * a.heads + head;
  float* q_s = smem;                        // [dim][CC]
  float* S_s = q_s + dim * CC;              // [dim][OV]
  float* u_s = S_s + dim * OV;              // [CC][OV]
  float* b_s = u_s + CC * OV;               // [CC][BP]: B with its rows (tokens) innermost
  for (int i = tid; i < dim * CC / 4; i += OT)
    cp_async16(q_s + 4 * i, a.YQ + (unit * dim + i / (CC / 4)) * 2 * CC + CC + 4 * (i % (CC / 4)));
  auto bring = [&](float* dst, const float* src, int rows) {      // rows x OV columns from colb on, zeros beyond the values
    for (int i = tid; i < rows * OV / 4; i += OT) {
      const int r = i / (OV / 4), c = 4 * (i % (OV / 4));
      const float* at = src + (size_t)r * vdim + colb + c;
      if (vdim % 4 == 0 && colb + c < vdim) cp_async16(dst + 4 * i, at);
      else
        for (int k = 0; k < 4; ++k) dst[4 * i + k] = colb + c + k < vdim ? at[k] : 0.f;
    }
  };
  bring(S_s, a.S + unit * dim * vdim, dim);
  bring(u_s, a.U + unit * CC * vdim, CC);
  for (int i = tid; i < CC * CC; i += OT) b_s[(i % CC) * BP + i / CC] = a.B[unit * CC * CC + i];
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  const int ty = tid / (OV / 4), tx = tid % (OV / 4);
  float o[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[i][c] = 0.f;
  auto mac = [&](const float* rows, int pitch, const float* cols, int depth) {
#pragma unroll 8
    for (int d = 0; d < depth; ++d) {
      const float4 r4 = *reinterpret_cast<const float4*>(rows + d * pitch + 4 * ty), c4 = *reinterpret_cast<const float4*>(cols + d * OV + 4 * tx);
      const float r[4] = {r4.x, r4.y, r4.z, r4.w}, c[4] = {c4.x, c4.y, c4.z, c4.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = fmaf(r[i], c[j], o[i][j]);
    }
  };
  mac(q_s, CC, S_s, dim);
  mac(b_s, BP, u_s, min(CC, 4 * ty + 4));      // B is zero beyond the diagonal
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = 4 * ty + i, col = colb + 4 * tx;
    if (t >= n) continue;
    float* dst = a.out + (size_t)(c0 + t) * a.out_stride + (size_t)head * vdim + col;
    if (vdim % 4 == 0 && (uintptr_t)dst % 16 == 0) {
      if (col < vdim) *reinterpret_cast<float4*>(dst) = make_float4(o[i][0], o[i][1], o[i][2], o[i][3]);
      continue;
    }
#pragma unroll
    for (int c = 0; c < 4; ++c)
      if (col + c < vdim) dst[c] = o[i][c];
  }
}

template <bool CH>
int launch_chunks(const PrepArgs& p, const WalkArgs& w, const OutArgs& o, int n_tokens, int dtype, cudaStream_t stream) {
  const int chunks = n_tokens / CC + p.n_entries;
  const size_t smem = prepare_floats(p.dim, CH) * sizeof(float);
  int rc = dispatch_dtype(dtype, [&](auto* tag) {
    using T = LLMK_ELEM(tag);
    if (smem > 48 * 1024) cudaFuncSetAttribute(delta_prepare_kernel<T, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_kernel(delta_prepare_kernel<T, CH>, dim3(chunks, p.heads), dim3(PT), smem, stream, p);
    LLMK_LAUNCH_CHECK("delta_prepare");
  });
  if (rc) return rc;
  if (p.dim <= 32) rc = launch_walk_of<32, CH>(w, p.n_entries, stream);
  else if (p.dim <= 64) rc = launch_walk_of<64, CH>(w, p.n_entries, stream);
  else if (p.dim <= 128) rc = launch_walk_of<128, CH>(w, p.n_entries, stream);
  else rc = launch_walk_of<256, CH>(w, p.n_entries, stream);
  if (rc) return rc;
  const size_t osmem = ((size_t)p.dim * (CC + OV) + CC * OV + CC * BP) * sizeof(float);
  if (osmem > 48 * 1024) cudaFuncSetAttribute(delta_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)osmem);
  launch_kernel(delta_chunk_out_kernel, dim3(chunks, p.heads, (p.vdim + OV - 1) / OV), dim3(OT), osmem, stream, o);
  LLMK_LAUNCH_CHECK("delta_chunk_out");
}

}  // namespace

// q, k [T, qk_heads * dim] (one row stride), v [T, heads * vdim] and b [T, heads] in the projections' kind; per_channel 0: a
// [T, heads] of the same kind, dt_bias float32 [heads]; else a float32 [T, heads * dim], dt_bias [heads * dim]; a_log float32
// [heads]; state float32, slot s at state + s * slot_stride holding [heads, dim, vdim]; out float32 [T, heads * vdim].  q is
// scaled by q_scale after its unit norm; norm_eps is added to the sums of squares.
LLMK_API int llmk_delta_scan(float* out, long long out_stride, const void* q, const void* k, long long qk_stride, const void* v,
                             long long v_stride, const void* b, long long b_stride, const void* a, long long a_stride,
                             const float* a_log, const float* dt_bias, float* state, long long slot_stride, const int* state_slots,
                             const int* cu_tokens, int n_entries, int heads, int qk_heads, int dim, int vdim, float q_scale,
                             float norm_eps, int per_channel, int dtype, cudaStream_t stream) {
  if (n_entries == 0) return 0;
  LLMK_REQUIRE(dim > 0 && dim <= 256, "delta_scan: key size %d (1 to 256)", dim);
  LLMK_REQUIRE(qk_heads > 0 && heads % qk_heads == 0 && vdim > 0, "delta_scan: %d heads do not divide into %d key heads", heads, qk_heads);
  LLMK_REQUIRE(n_entries <= 65535 && heads <= 65535, "delta_scan: too many entries or heads for one launch");
  DeltaArgs args = {out, out_stride, q, k, qk_stride, v, v_stride, b, a, b_stride, a_stride, a_log, dt_bias, state, slot_stride,
                    state_slots, cu_tokens, heads, qk_heads, dim, vdim, q_scale, norm_eps};
  return dispatch_dtype(dtype, [&](auto* tag) {
    using T = LLMK_ELEM(tag);
    return per_channel ? launch_delta_of<T, true>(args, n_entries, stream) : launch_delta_of<T, false>(args, n_entries, stream);
  });
}

// The same rule for a step with prompt portions, chunk by chunk (see delta_prepare_kernel).  n_tokens: the step's tokens.
// Float32 scratch for n_tokens / 32 + n_entries chunks of every head: YQ (dim * 64 floats a chunk and head), K (32 * dim),
// W (32 * vdim), B (32 * 32), G (1; per_channel: dim), S (dim * vdim).
LLMK_API int llmk_delta_chunk_scan(float* out, long long out_stride, const void* q, const void* k, long long qk_stride,
                                   const void* v, long long v_stride, const void* b, long long b_stride, const void* a,
                                   long long a_stride, const float* a_log, const float* dt_bias, float* state, long long slot_stride,
                                   const int* state_slots, const int* cu_tokens, int n_entries, int n_tokens, int heads,
                                   int qk_heads, int dim, int vdim, float q_scale, float norm_eps, int per_channel, float* YQ, float* K,
                                   float* W, float* B, float* G, float* S, int dtype, cudaStream_t stream) {
  if (n_entries == 0 || n_tokens == 0) return 0;
  LLMK_REQUIRE(dim > 0 && dim <= 256, "delta_chunk_scan: key size %d (1 to 256)", dim);
  LLMK_REQUIRE(qk_heads > 0 && heads % qk_heads == 0 && vdim > 0, "delta_chunk_scan: %d heads do not divide into %d key heads", heads, qk_heads);
  LLMK_REQUIRE(n_entries <= 65535 && heads <= 65535, "delta_chunk_scan: too many entries or heads for one launch");
  LLMK_REQUIRE(YQ && K && W && B && G && S, "delta_chunk_scan: the scratch is missing");
  const PrepArgs p = {q, k, qk_stride, v, v_stride, b, a, b_stride, a_stride, a_log, dt_bias, cu_tokens, n_entries, heads, qk_heads, dim,
                      vdim, q_scale, norm_eps, YQ, K, W, B, G,
                      dim % 4 == 0 && qk_stride % 4 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)k % 16 == 0 &&
                          (!per_channel || (a_stride % 4 == 0 && (uintptr_t)a % 16 == 0 && (uintptr_t)dt_bias % 16 == 0))};
  const WalkArgs w = {YQ, K, G, W, S, state, slot_stride, state_slots, cu_tokens, heads, dim, vdim};
  const OutArgs o = {out, out_stride, YQ, B, W, S, cu_tokens, n_entries, heads, dim, vdim};
  return per_channel ? launch_chunks<true>(p, w, o, n_tokens, dtype, stream) : launch_chunks<false>(p, w, o, n_tokens, dtype, stream);
}
