// RMS norms on both sides of a residual sum, for blocks that norm a sublayer's input and its output:
//
//     resid += mult * rms(delta) * post            (post null: resid += mult * delta)
//     out    = rms(resid) * pre                    (out null: nothing more)
//
// with rms(x) = x / sqrt(mean(x^2) + eps), in one pass over the row, everything float32.  delta is what the sublayer left, and
// may be left before its last sums, which then need no kernel and no buffer of their own:
//
//     delta[t] = sa * a[t] + bias                                              a product's rows (a tensor or its split-K partial
//              + sb * gate[t] * b[t]                                           results) and its bias; a second such product;
//              + sum_j weights[t, j] * (slot[t, j] >= 0 ? y[slot[t, j]]        the rows of a routed feed-forward, summed in the
//                                       : ids[t, j] >= first ? x[t] : 0)       order of j, identity experts as in routed.cu
//
// each term optional.  A CTA per row; rows of up to 8192 elements on the 8-grid stay in registers.
#include "common.cuh"

namespace {

template <typename T>
struct Delta {
  MaybePartial<T> a; float sa; const float* bias;
  MaybePartial<T> b; float sb; const float* gate;
  const float* y; const int *slots, *ids; const float* weights; int top, first;
  const T* x; long long x_stride;

  __host__ __device__ bool present() const { return a.direct || a.parts || y; }
  // eight consecutive columns from c on (VEC), or one
  template <bool VEC>
  __device__ __forceinline__ void at(int t, int c, int hidden, float* d) const {
    constexpr int N = VEC ? 8 : 1;
    const size_t i = (size_t)t * hidden + c;
#pragma unroll
    for (int k = 0; k < N; ++k) d[k] = 0.f;
    auto add = [&](const MaybePartial<T>& m, float s) {
      float v[N];
      if constexpr (VEC) m.at8(i, v); else v[0] = m.at(i);
#pragma unroll
      for (int k = 0; k < N; ++k) d[k] = fmaf(s, v[k], d[k]);
    };
    if (a.present()) add(a, sa);
    if (bias) {
      float v[N];
      if constexpr (VEC) Vec8<float>::load(bias + c, v); else v[0] = bias[c];
#pragma unroll
      for (int k = 0; k < N; ++k) d[k] += v[k];
    }
    if (y) {
#pragma unroll 4
      for (int j = 0; j < top; ++j) {
        const int slot = slots[(size_t)t * top + j];
        const float w = weights[(size_t)t * top + j];
        float v[N];
        if (slot >= 0) {
          const float* src = y + (size_t)slot * hidden + c;
          if constexpr (VEC) Vec8<float>::load(src, v); else v[0] = *src;
        } else if (ids && ids[(size_t)t * top + j] >= first) {
          const T* src = x + (size_t)t * x_stride + c;
          if constexpr (VEC) Vec8<T>::load(src, v); else v[0] = to_f32(*src);
        } else {
          continue;
        }
#pragma unroll
        for (int k = 0; k < N; ++k) d[k] = fmaf(w, v[k], d[k]);
      }
    }
    if (b.present()) add(b, gate ? sb * gate[t] : sb);
  }
  bool vector_ok() const {
    return a.vector_ok() && b.vector_ok() && (uintptr_t)bias % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)x % 16 == 0 && x_stride % 8 == 0;
  }
};

// NV > 0: the row in registers, NV vectors of eight per thread; 0: any rows, in shared memory.
template <typename T, int NV>
__global__ void __launch_bounds__(256)
sandwich_norms_kernel(float* resid, Delta<T> delta, const float* __restrict__ post, float mult, const float* __restrict__ pre,
                      T* out, int hidden, float eps) {
  extern __shared__ float row_s[];
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const size_t base = (size_t)t * hidden;
  const bool has = delta.present();
  auto rstd = [&](float ss) { return 1.f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps); };
  if constexpr (NV > 0) {
    float r[NV][8];
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int c = (v * 256 + threadIdx.x) * 8;
      if (c < hidden) Vec8<float>::load(resid + base + c, r[v]);
    }
    if (has) {
      float y[NV][8], ss = 0.f;
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int c = (v * 256 + threadIdx.x) * 8;
        if (c >= hidden) continue;
        delta.template at<true>(t, c, hidden, y[v]);
#pragma unroll
        for (int k = 0; k < 8; ++k) ss = fmaf(y[v][k], y[v][k], ss);
      }
      const float f = post ? mult * rstd(ss) : mult;
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int c = (v * 256 + threadIdx.x) * 8;
        if (c >= hidden) continue;
        float w[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
        if (post) Vec8<float>::load(post + c, w);
#pragma unroll
        for (int k = 0; k < 8; ++k) r[v][k] = fmaf(f * y[v][k], w[k], r[v][k]);
        Vec8<float>::store(resid + base + c, r[v]);
      }
    }
    if (!out) return;
    float ss = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      if ((v * 256 + threadIdx.x) * 8 >= hidden) continue;
#pragma unroll
      for (int k = 0; k < 8; ++k) ss = fmaf(r[v][k], r[v][k], ss);
    }
    const float f = rstd(ss);
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int c = (v * 256 + threadIdx.x) * 8;
      if (c >= hidden) continue;
      float w[8];
      Vec8<float>::load(pre + c, w);
#pragma unroll
      for (int k = 0; k < 8; ++k) w[k] *= f * r[v][k];
      Vec8<T>::store(out + base + c, w);
    }
  } else {
    if (has) {
      float ss = 0.f;
      for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        float y;
        delta.template at<false>(t, c, hidden, &y);
        row_s[c] = y;
        ss = fmaf(y, y, ss);
      }
      const float f = post ? mult * rstd(ss) : mult;
      for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const float r = fmaf(f * row_s[c], post ? post[c] : 1.f, resid[base + c]);
        resid[base + c] = r;
        row_s[c] = r;
      }
    } else {
      for (int c = threadIdx.x; c < hidden; c += blockDim.x) row_s[c] = resid[base + c];
    }
    if (!out) return;
    float ss = 0.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) ss = fmaf(row_s[c], row_s[c], ss);
    const float f = rstd(ss);
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) out[base + c] = from_f32<T>(row_s[c] * f * pre[c]);
  }
}

}  // namespace

// a / a_parts, b / b_parts: a tensor [rows, hidden] of the element kind or float32 partial results [splits][rows][hidden], or
// neither; bias float32 [hidden] or null; gate float32 [rows] or null.  y float32 [slots, hidden] with slots, weights [rows, top]
// (and ids, first, x [rows, x_stride] where there are identity experts), or null.  post, pre float32 [hidden] or null; out
// [rows, hidden] of the element kind or null (then pre is not read); out may be x (a row is read before it is written).
LLMK_API int llmk_sandwich_norms(float* resid, const void* a, const float* a_parts, int a_splits, long long a_stride, float sa,
                                 const float* bias, const void* b, const float* b_parts, int b_splits, long long b_stride, float sb,
                                 const float* gate, const float* y, const int* slots, const float* weights, int top, const int* ids,
                                 int first, const void* x, long long x_stride, const float* post, float mult, const float* pre,
                                 void* out, int rows, int hidden, float eps, int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  LLMK_REQUIRE(!(a && a_parts) && !(b && b_parts), "sandwich_norms: a term is a tensor or partial results, not both");
  LLMK_REQUIRE(out == nullptr || pre != nullptr, "sandwich_norms: an output needs its weight");
  LLMK_REQUIRE(y == nullptr || (slots && weights && top > 0 && (!ids || x)), "sandwich_norms: weighted rows lack their slots, weights or inputs");
  const size_t smem = (size_t)hidden * sizeof(float);
  LLMK_REQUIRE(smem <= 200 * 1024, "sandwich_norms: rows of %d elements exceed the shared memory", hidden);
  return dispatch_dtype(dtype, [&](auto* tag) {
    using T = LLMK_ELEM(tag);
    const Delta<T> d{{(const T*)a, a_parts, a_splits, a_stride}, sa, bias, {(const T*)b, b_parts, b_splits, b_stride}, sb, gate,
                     y, slots, ids, weights, top, first, (const T*)x, x_stride};
    const bool vec = hidden % 8 == 0 && hidden <= 8192 && d.vector_ok() && (uintptr_t)resid % 16 == 0 && (uintptr_t)post % 16 == 0 &&
                     (uintptr_t)pre % 16 == 0 && (uintptr_t)out % 16 == 0;
    auto go = [&](auto kern, size_t bytes) {
      if (bytes > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
      launch_kernel(kern, dim3(rows), dim3(256), bytes, stream, resid, d, post, mult, pre, (T*)out, hidden, eps);
    };
    if (vec && hidden <= 2048) go(sandwich_norms_kernel<T, 1>, 0);
    else if (vec && hidden <= 4096) go(sandwich_norms_kernel<T, 2>, 0);
    else if (vec) go(sandwich_norms_kernel<T, 4>, 0);
    else go(sandwich_norms_kernel<T, 0>, smem);
    LLMK_LAUNCH_CHECK("sandwich_norms");
  });
}
