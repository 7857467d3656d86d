// Attention over a latent cache whose rows are wider than the tcgen05 kernels take (bfloat16, 192 to 640 channels in steps of 64):
// one vector per token is key and value of every head, so the queries of all heads of a request meet the same rows.
//
// The rows of the query matrix are (token, head) pairs as they lie in memory, [n_tokens * heads, W]; a CTA of eight warps takes 64
// or 16 of them (RG groups of 16) and walks over its request's keys in tiles of KT rows, which serve both products:
//     S = Q C^T    a warp makes 16 rows x KT / KG keys           (KG = 8 / RG warps share a group of rows)
//     O += P C     a warp makes 16 rows x W / KG columns
// so no part of either product is made twice; P passes through shared memory between the two, as bfloat16, and the running
// maximum of a row is agreed on by its KG warps there.  Tiles arrive by asynchronous 16-byte copies through the block table,
// STAGES deep.  Operands come from shared memory by ldmatrix into warp-level MMAs (mma.sync): the accumulator of 64 x 640
// float32 numbers fits the registers of eight warps, and what bounds the kernel is reading the tile from shared memory.
// Scores, softmax and sums are float32.
//
// Steps of single tokens split the keys over gridDim.y ranges (the results of the ranges are merged by wide_merge_kernel);
// steps with prompt portions run one range, heaviest tiles first.
#include "common.cuh"

namespace {

using bf16 = __nv_bfloat16;
constexpr int WARPS = 8, THREADS = WARPS * 32, PAD = 8;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldsm2_t(uint32_t (&r)[2], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
  const int bytes = valid ? 16 : 0;                        // the rest of the 16 bytes is filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int NB, int RG>
struct Wide {
  static constexpr int W = NB * 64, KG = WARPS / RG, KT = RG == 1 ? 64 : 32, KW = KT / KG, PITCH = W + PAD, P_PITCH = KT + PAD;
  static constexpr int ROWS = 16 * RG, COLS = W / KG, STAGES = RG == 1 ? 2 : (NB <= 6 ? 3 : 2);
  static constexpr size_t SMEM = ((size_t)(ROWS + STAGES * KT) * PITCH + (size_t)ROWS * P_PITCH) * sizeof(bf16);
};

struct WideArgs {
  bf16* out; const bf16* q; const bf16* pages;
  const int* block_table; int table_width;
  const int *cu_tokens, *kv_lens;
  int n_entries, heads, page_size, width;
  float scale_log2e;
  int splits; float *part_o, *part_ml;          // ranges > 1: [rows of the step, splits, W] and [.., splits, 2]
};

template <int NB, int RG>
__global__ void __launch_bounds__(THREADS, 1)
attention_wide_kernel(WideArgs a) {
  using C = Wide<NB, RG>;
  constexpr int W = C::W, KG = C::KG, KT = C::KT, KW = C::KW, PITCH = C::PITCH, P_PITCH = C::P_PITCH, ROWS = C::ROWS, COLS = C::COLS,
                STAGES = C::STAGES, NT = KW / 8, OT = COLS / 8;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ float red_s[KG][ROWS];
  pdl_launch_dependents();
  pdl_wait();
  bf16* q_s = reinterpret_cast<bf16*>(smem_raw);             // [ROWS][PITCH]
  bf16* c_s = q_s + ROWS * PITCH;                            // [STAGES][KT][PITCH]
  bf16* p_s = c_s + STAGES * KT * PITCH;                     // [ROWS][P_PITCH]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rg = warp / KG, kg = warp % KG;
  // the tile: rows of one entry.  Tiles are numbered from the step's end, so that the ones with most keys start first
  int idx = gridDim.x - 1 - blockIdx.x, entry = -1, row0 = 0, n_rows = 0;
  for (int e = 0; e < a.n_entries; ++e) {
    const int rows = (a.cu_tokens[e + 1] - a.cu_tokens[e]) * a.heads, tiles = (rows + ROWS - 1) / ROWS;
    if (idx < tiles) { entry = e; row0 = a.cu_tokens[e] * a.heads + idx * ROWS; n_rows = min(ROWS, rows - idx * ROWS); break; }
    idx -= tiles;
  }
  if (entry < 0) return;
  const int held = min(a.kv_lens[entry], a.table_width * a.page_size);
  const int first_pos = held - (a.cu_tokens[entry + 1] - a.cu_tokens[entry]);      // position of the entry's first token of this step
  auto pos_of = [&](int r) { return first_pos + (row0 + r) / a.heads - a.cu_tokens[entry]; };      // r < n_rows
  const int n_keys = min(held, pos_of(n_rows - 1) + 1);
  int k_begin = 0, k_end = n_keys;
  if (a.splits > 1) {
    int range = (n_keys + a.splits - 1) / a.splits;
    range = (range + KT - 1) / KT * KT;
    k_begin = blockIdx.y * range;
    k_end = min(n_keys, k_begin + range);
  }
  const int* table = a.block_table + (size_t)entry * a.table_width;
  constexpr int CH = W / 8;                                  // 16-byte pieces of a row
  for (int i = tid; i < ROWS * CH; i += THREADS) {
    const int r = i / CH, c = (i % CH) * 8;
    cp_async16(q_s + r * PITCH + c, a.q + (size_t)(row0 + min(r, n_rows - 1)) * W + c, r < n_rows);
  }
  auto stage_tile = [&](int t) {                             // keys k_begin + t * KT ..
    bf16* dst = c_s + (t % STAGES) * KT * PITCH;
    const int k0 = k_begin + t * KT;
    for (int i = tid; i < KT * CH; i += THREADS) {
      const int kl = i / CH, c = (i % CH) * 8, k = k0 + kl;
      const bool valid = k < k_end;
      const int kq = valid ? k : k_begin;
      const size_t row = (size_t)table[kq / a.page_size] * a.page_size + kq % a.page_size;
      cp_async16(dst + kl * PITCH + c, a.pages + row * W + c, valid);
    }
  };
  const int n_tiles = k_begin < k_end ? (k_end - k_begin + KT - 1) / KT : 0;
#pragma unroll
  for (int t = 0; t < STAGES - 1; ++t) {
    if (t < n_tiles) stage_tile(t);
    cp_async_commit();
  }
  const int ra = rg * 16 + (lane >> 2), rb = ra + 8;         // the lane's two rows
  const int pa = ra < n_rows ? pos_of(ra) : -1, pb = rb < n_rows ? pos_of(rb) : -1;
  float o[OT][4];
#pragma unroll
  for (int i = 0; i < OT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float ma = -INFINITY, mb = -INFINITY, la = 0.f, lb = 0.f;  // l: this lane's share of this warp's keys
  const bf16* q_at = q_s + (rg * 16 + (lane & 15)) * PITCH + ((lane >> 4) << 3);

  for (int t = 0; t < n_tiles; ++t) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();                                         // tile t has landed, and everyone is done with the tile before it
    if (t + STAGES - 1 < n_tiles) stage_tile(t + STAGES - 1);
    cp_async_commit();
    const bf16* tile = c_s + (t % STAGES) * KT * PITCH;
    // ---- S: 16 rows x KW keys
    float s[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    if constexpr (NT == 2) {
      const bf16* k_at = tile + (kg * KW + (lane & 7) + ((lane >> 4) << 3)) * PITCH + (((lane >> 3) & 1) << 3);
#pragma unroll 4
      for (int x = 0; x < W; x += 16) {
        uint32_t qa[4], kb[4];
        ldsm4(qa, q_at + x);
        ldsm4(kb, k_at + x);
        mma(s[0], qa, kb[0], kb[1]);
        mma(s[1], qa, kb[2], kb[3]);
      }
    } else {
      static_assert(NT == 1 || NT == 2, "a warp scores 8 or 16 keys of a tile");
      const bf16* k_at = tile + (kg * KW + (lane & 7)) * PITCH + ((lane >> 3) << 3);
#pragma unroll 2
      for (int x = 0; x < W; x += 32) {
        uint32_t qa[4], qb[4], kb[4];
        ldsm4(qa, q_at + x);
        ldsm4(qb, q_at + x + 16);
        ldsm4(kb, k_at + x);
        mma(s[0], qa, kb[0], kb[1]);
        mma(s[0], qb, kb[2], kb[3]);
      }
    }
    // ---- scale, mask, the row's maximum over the tile
    float ta = -INFINITY, tb = -INFINITY;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int k = k_begin + t * KT + kg * KW + i * 8 + 2 * (lane & 3) + j;
        s[i][j] = k < k_end && k <= pa ? s[i][j] * a.scale_log2e : -INFINITY;
        s[i][2 + j] = k < k_end && k <= pb ? s[i][2 + j] * a.scale_log2e : -INFINITY;
        ta = fmaxf(ta, s[i][j]);
        tb = fmaxf(tb, s[i][2 + j]);
      }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      ta = fmaxf(ta, __shfl_xor_sync(0xffffffffu, ta, x));
      tb = fmaxf(tb, __shfl_xor_sync(0xffffffffu, tb, x));
    }
    if ((lane & 3) == 0) { red_s[kg][ra] = ta; red_s[kg][rb] = tb; }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < KG; ++x) { ta = fmaxf(ta, red_s[x][ra]); tb = fmaxf(tb, red_s[x][rb]); }
    const float na = fmaxf(ma, ta), nb = fmaxf(mb, tb);
    const float ua = na == -INFINITY ? 0.f : na, ub = nb == -INFINITY ? 0.f : nb;      // a row without a visible key so far
    const float fa = ex2(ma - ua), fb = ex2(mb - ub);        // 0 while the old maximum is -inf
    const bool moved = na != ma || nb != mb;
    ma = na; mb = nb;
    la *= fa; lb *= fb;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const float p0 = ex2(s[i][0] - ua), p1 = ex2(s[i][1] - ua), p2 = ex2(s[i][2] - ub), p3 = ex2(s[i][3] - ub);
      la += p0 + p1;
      lb += p2 + p3;
      bf16* at = p_s + ra * P_PITCH + kg * KW + i * 8 + 2 * (lane & 3);
      *reinterpret_cast<__nv_bfloat162*>(at) = __floats2bfloat162_rn(p0, p1);
      *reinterpret_cast<__nv_bfloat162*>(at + 8 * P_PITCH) = __floats2bfloat162_rn(p2, p3);
    }
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int i = 0; i < OT; ++i) { o[i][0] *= fa; o[i][1] *= fa; o[i][2] *= fb; o[i][3] *= fb; }
    }
    __syncthreads();                                         // P is complete
    // ---- O += P C: 16 rows x COLS columns
#pragma unroll
    for (int k0 = 0; k0 < KT; k0 += 16) {
      uint32_t p[4];
      ldsm4(p, p_s + (rg * 16 + (lane & 15)) * P_PITCH + k0 + ((lane >> 4) << 3));
      const bf16* v_at = tile + (k0 + (lane & 15)) * PITCH + kg * COLS;
#pragma unroll
      for (int i = 0; i + 1 < OT; i += 2) {
        uint32_t b[4];
        ldsm4_t(b, v_at + i * 8 + ((lane >> 4) << 3));
        mma(o[i], p, b[0], b[1]);
        mma(o[i + 1], p, b[2], b[3]);
      }
      if constexpr (OT % 2 == 1) {
        uint32_t b[2];
        ldsm2_t(b, v_at + (OT - 1) * 8);
        mma(o[OT - 1], p, b[0], b[1]);
      }
    }
  }
  cp_async_wait<0>();
  // ---- the rows' sums over their KG warps
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    la += __shfl_xor_sync(0xffffffffu, la, x);
    lb += __shfl_xor_sync(0xffffffffu, lb, x);
  }
  __syncthreads();
  if ((lane & 3) == 0) { red_s[kg][ra] = la; red_s[kg][rb] = lb; }
  __syncthreads();
  la = lb = 0.f;
#pragma unroll
  for (int x = 0; x < KG; ++x) { la += red_s[x][ra]; lb += red_s[x][rb]; }
  if (a.splits > 1) {
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = h ? rb : ra;
      if (r >= n_rows) continue;
      const size_t at = (size_t)(row0 + r) * a.splits + blockIdx.y;
      if (kg == 0 && (lane & 3) == 0) { a.part_ml[at * 2] = h ? mb : ma; a.part_ml[at * 2 + 1] = h ? lb : la; }
      if (n_tiles == 0) continue;                            // an empty range: its weight in the merge is zero
#pragma unroll
      for (int i = 0; i < OT; ++i)
        *reinterpret_cast<float2*>(a.part_o + at * W + kg * COLS + i * 8 + 2 * (lane & 3)) = make_float2(o[i][2 * h], o[i][2 * h + 1]);
    }
    return;
  }
  const float ia = la > 0.f ? 1.f / la : 0.f, ib = lb > 0.f ? 1.f / lb : 0.f;
#pragma unroll
  for (int i = 0; i < OT; ++i) {
    const int c = kg * COLS + i * 8 + 2 * (lane & 3);
    if (ra < n_rows) *reinterpret_cast<__nv_bfloat162*>(a.out + (size_t)(row0 + ra) * W + c) = __floats2bfloat162_rn(o[i][0] * ia, o[i][1] * ia);
    if (rb < n_rows) *reinterpret_cast<__nv_bfloat162*>(a.out + (size_t)(row0 + rb) * W + c) = __floats2bfloat162_rn(o[i][2] * ib, o[i][3] * ib);
  }
}

// The ranges of a row merged in their order.  One CTA per row.
__global__ void __launch_bounds__(128)
wide_merge_kernel(bf16* __restrict__ out, const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits, int width) {
  __shared__ float w_s[64];
  pdl_launch_dependents();
  pdl_wait();
  const size_t base = (size_t)blockIdx.x * splits;
  if (threadIdx.x < 32) {
    float m = -INFINITY;
    for (int s = threadIdx.x; s < splits; s += 32) m = fmaxf(m, part_ml[(base + s) * 2]);
    m = warp_max(m);
    float l = 0.f;
    for (int s = threadIdx.x; s < splits; s += 32) {
      const float ms = part_ml[(base + s) * 2], f = ms > -INFINITY ? ex2(ms - m) : 0.f;
      w_s[s] = f;
      l += f * part_ml[(base + s) * 2 + 1];
    }
    l = warp_sum(l);
    const float inv = l > 0.f ? 1.f / l : 0.f;
    for (int s = threadIdx.x; s < splits; s += 32) w_s[s] *= inv;
  }
  __syncthreads();
  for (int c = threadIdx.x * 4; c < width; c += 128 * 4) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
      const float w = w_s[s];
      if (w == 0.f) continue;
      const float4 v = *reinterpret_cast<const float4*>(part_o + (base + s) * width + c);
      acc.x = fmaf(w, v.x, acc.x); acc.y = fmaf(w, v.y, acc.y); acc.z = fmaf(w, v.z, acc.z); acc.w = fmaf(w, v.w, acc.w);
    }
    __nv_bfloat162* dst = reinterpret_cast<__nv_bfloat162*>(out + (size_t)blockIdx.x * width + c);
    dst[0] = __floats2bfloat162_rn(acc.x, acc.y);
    dst[1] = __floats2bfloat162_rn(acc.z, acc.w);
  }
}

template <int NB, int RG>
int launch_wide(const WideArgs& a, int n_tokens, cudaStream_t stream) {
  using C = Wide<NB, RG>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attention_wide_kernel<NB, RG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM);
    if (e != cudaSuccess) return llmk_fail((int)e, "attention_wide: cannot set %d bytes of shared memory: %s", (int)C::SMEM, cudaGetErrorString(e));
    configured = true;
  }
  // tiles of any step of so many tokens and entries: what is not needed leaves at once
  const long long tiles = (long long)n_tokens * a.heads / C::ROWS + a.n_entries;
  LLMK_REQUIRE(tiles <= 0x7fffffffLL, "attention_wide: too many rows for one launch");
  launch_kernel(attention_wide_kernel<NB, RG>, dim3((unsigned)tiles, a.splits), dim3(THREADS), C::SMEM, stream, a);
  if (a.splits > 1)
    launch_kernel(wide_merge_kernel, dim3((unsigned)(n_tokens * a.heads)), dim3(128), 0, stream, a.out, (const float*)a.part_o,
                  (const float*)a.part_ml, a.splits, a.width);
  LLMK_LAUNCH_CHECK("attention_wide");
}

}  // namespace

// q, out [n_tokens, heads * width] bfloat16 contiguous; pages [pages, 1, page_size, width]; entry e's tokens are rows
// cu_tokens[e] .. of q, its keys (the new tokens' included) number kv_lens[e]; a token sees the keys up to its own.  width: 192, 256,
// 320, 384, 512, 576 or 640.  small: tiles of 16 rows (steps of single tokens with few heads), else 64.  splits > 1: part_o float32
// [n_tokens * heads, splits, width] and part_ml [.., splits, 2].
LLMK_API int llmk_attention_wide(void* out, const void* q, const void* pages, const int* block_table, int table_width,
                                 const int* cu_tokens, const int* kv_lens, int n_tokens, int n_entries, int heads, int width,
                                 int page_size, float scale, int small, int splits, float* part_o, float* part_ml, cudaStream_t stream) {
  if (n_tokens == 0 || n_entries == 0) return 0;
  LLMK_REQUIRE(heads > 0 && page_size > 0, "attention_wide: bad sizes");
  LLMK_REQUIRE(splits >= 1 && splits <= 64 && (splits == 1 || (part_o && part_ml)), "attention_wide: %d ranges (1 to 64) need their scratch", splits);
  LLMK_REQUIRE((uintptr_t)q % 16 == 0 && (uintptr_t)out % 4 == 0 && (uintptr_t)pages % 16 == 0 && (uintptr_t)part_o % 16 == 0,
               "attention_wide: operands off the 16-byte grid");
  const WideArgs a{(bf16*)out, (const bf16*)q, (const bf16*)pages, block_table, table_width, cu_tokens, kv_lens, n_entries, heads, page_size, width,
                   scale * 1.4426950408889634f, splits, part_o, part_ml};
#define LLMK_WIDE(NB) case NB * 64: return small ? launch_wide<NB, 1>(a, n_tokens, stream) : launch_wide<NB, 4>(a, n_tokens, stream)
  switch (width) {
    LLMK_WIDE(3);
    LLMK_WIDE(4);
    LLMK_WIDE(5);
    LLMK_WIDE(6);
    LLMK_WIDE(8);
    LLMK_WIDE(9);
    LLMK_WIDE(10);
  }
#undef LLMK_WIDE
  return llmk_fail(-1, "attention_wide: rows of %d channels (192, 256, 320, 384, 512, 576 or 640)", width);
}
