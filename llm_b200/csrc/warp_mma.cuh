// Warp-level bfloat16 MMAs (mma.sync) and what goes with them: asynchronous copies into shared memory, operand loads from it,
// and a float32 operand as three bfloat16 numbers.  For products whose operands a warp makes itself in registers, on tiles too
// small for tensor memory.
#pragma once

#include "common.cuh"

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(void* smem_dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(smem_dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory"); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two float32 numbers as three pairs of bfloat16 numbers whose sums they are (to the last of their 24 bits or so).
__device__ __forceinline__ void split3(float x, float y, uint32_t (&p)[3]) {
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    p[i] = *reinterpret_cast<const uint32_t*>(&h);
    x -= __low2float(h); y -= __high2float(h);
  }
}

// rows [0, n) of a [.., cols] tensor into shared memory with pitch `pitch`, zeros in rows n .. ROWS and columns up to `cols_pad`
// (cols a multiple of 8, cols_pad of 8)
template <int ROWS, int THREADS>
__device__ __forceinline__ void bring_rows(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, long long stride, int n, int cols, int cols_pad) {
  const int per = cols_pad / 8;
  for (int i = threadIdx.x; i < ROWS * per; i += THREADS) {
    const int r = i / per, c = (i % per) * 8;
    __nv_bfloat16* at = dst + r * pitch + c;
    if (r < n && c < cols) cp_async16(at, src + (size_t)r * stride + c);
    else *reinterpret_cast<uint4*>(at) = make_uint4(0, 0, 0, 0);
  }
}
