// The norm behind a sum, for layers whose sublayers read the residual stream itself:
//
//   x <- n(alpha x + c_1 (y_1 + b_1) [+ c_2 (y_2 + b_2)])        x float32, in place
//   n(v) = v / sqrt(mean(v^2) + eps) * w                         (w null: x is the sum itself)
//   out  = x in another dtype                                    (out given: the next sublayer reads it)
//
// A term y is a matrix in float32 or bfloat16, or the float32 partial sums [splits, rows, hidden] of a K-split
// product, added here in split order; b is a float32 vector along the row or null.  Everything is float32.
// One block per row; the order of a row's additions depends on hidden and the block's size only.
#include "common.cuh"

namespace ifx {

struct SumTerm {
  const void* y;             // null: no term
  int is_bf16, splits;
  size_t split_stride;
  float c;
  const float* bias;
};

template <int V> struct FloatVec;
template <> struct FloatVec<1> { using type = float; };
template <> struct FloatVec<4> { using type = float4; };

template <int V>
__device__ __forceinline__ void load_vec(float (&v)[V], const float* p) {
  *reinterpret_cast<typename FloatVec<V>::type*>(v) = *reinterpret_cast<const typename FloatVec<V>::type*>(p);
}

template <int V>
__device__ __forceinline__ void load_vec(float (&v)[V], const __nv_bfloat16* p) {
  if constexpr (V == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  } else {
    v[0] = __bfloat162float(*p);
  }
}

template <int V>
__device__ __forceinline__ void store_vec(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const uint32_t*>(&a);
    raw.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

template <int V>
__device__ __forceinline__ void add_term(float (&acc)[V], const SumTerm& t, size_t at, int col) {
  if (t.y == nullptr) return;
  float s[V];
  if (t.is_bf16) {
    load_vec<V>(s, reinterpret_cast<const __nv_bfloat16*>(t.y) + at);
  } else {
    const float* p = reinterpret_cast<const float*>(t.y) + at;
    load_vec<V>(s, p);
    for (int k = 1; k < t.splits; k += 4) {                  // four slices in flight, added in split order
      float part[4][V];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (k + j < t.splits) load_vec<V>(part[j], p + (size_t)(k + j) * t.split_stride);
        else
#pragma unroll
          for (int e = 0; e < V; ++e) part[j][e] = 0.0f;
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) s[e] += part[j][e];
    }
  }
  if (t.bias != nullptr) {
    float b[V];
    load_vec<V>(b, t.bias + col);
#pragma unroll
    for (int e = 0; e < V; ++e) s[e] += b[e];
  }
#pragma unroll
  for (int e = 0; e < V; ++e) acc[e] = fmaf(t.c, s[e], acc[e]);
}

template <int V>
__global__ void __launch_bounds__(1024) norm_of_sum_kernel(float* __restrict__ x, float alpha, const SumTerm t1, const SumTerm t2,
                                                           const float* __restrict__ w, float eps, void* __restrict__ out,
                                                           int out_is_bf16, int hidden) {
  extern __shared__ __align__(16) float row_s[];             // what of the row does not fit a thread's registers
  __shared__ float scratch[32];
  pdl_launch_dependents();
  const size_t base = (size_t)blockIdx.x * hidden;
  const int first = threadIdx.x * V;
  float wv[V];
#pragma unroll
  for (int e = 0; e < V; ++e) wv[e] = 1.0f;
  if (w != nullptr && first < hidden) load_vec<V>(wv, w + first);
  pdl_wait();
  float held[V];                                             // the thread's first elements
#pragma unroll
  for (int e = 0; e < V; ++e) held[e] = 0.0f;
  float ss = 0.0f;
  for (int i = first; i < hidden; i += blockDim.x * V) {
    float v[V];
    load_vec<V>(v, x + base + i);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] *= alpha;
    add_term<V>(v, t1, base + i, i);
    add_term<V>(v, t2, base + i, i);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
    if (i == first) {
#pragma unroll
      for (int e = 0; e < V; ++e) held[e] = v[e];
    } else {
      *reinterpret_cast<typename FloatVec<V>::type*>(row_s + i) = *reinterpret_cast<const typename FloatVec<V>::type*>(v);
    }
  }
  float inv = 1.0f;
  if (w != nullptr) {
    ss = block_sum(ss, scratch);
    inv = 1.0f / sqrtf(ss / (float)hidden + eps);
  }
  for (int i = first; i < hidden; i += blockDim.x * V) {
    float v[V];
    if (i == first) {
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = held[e] * inv * wv[e];
    } else {
      float wi[V];
#pragma unroll
      for (int e = 0; e < V; ++e) wi[e] = 1.0f;
      if (w != nullptr) load_vec<V>(wi, w + i);
      load_vec<V>(v, row_s + i);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = v[e] * inv * wi[e];
    }
    *reinterpret_cast<typename FloatVec<V>::type*>(x + base + i) = *reinterpret_cast<const typename FloatVec<V>::type*>(v);
    if (out != nullptr) {
      if (out_is_bf16) store_vec<V>(reinterpret_cast<__nv_bfloat16*>(out) + base + i, v);
      else *reinterpret_cast<typename FloatVec<V>::type*>(reinterpret_cast<float*>(out) + base + i) =
               *reinterpret_cast<const typename FloatVec<V>::type*>(v);
    }
  }
}

}  // namespace ifx

using namespace ifx;

// y1 (needed), y2 (may be null): dtype IFX_DT_*; splits >= 1 slices of [rows, hidden] (more than one: float32 only).
extern "C" int ifx_norm_of_sum(float* x, float alpha, const void* y1, int dtype1, int splits1, float c1, const float* bias1,
                               const void* y2, int dtype2, int splits2, float c2, const float* bias2, const float* w, float eps,
                               void* out, int out_dtype, int rows, int hidden, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (hidden <= 0 || y1 == nullptr || splits1 < 1 || (y2 != nullptr && splits2 < 1)) return IFX_E_BADARG;
  for (int dt : {dtype1, dtype2, out_dtype})
    if (dt != IFX_DT_F32 && dt != IFX_DT_BF16) return IFX_E_DTYPE;
  if ((dtype1 == IFX_DT_BF16 && splits1 > 1) || (y2 != nullptr && dtype2 == IFX_DT_BF16 && splits2 > 1)) return IFX_E_BADARG;
  const size_t stride = (size_t)rows * hidden;
  const SumTerm t1{y1, dtype1 == IFX_DT_BF16, splits1, stride, c1, bias1};
  const SumTerm t2{y2, dtype2 == IFX_DT_BF16, splits2, stride, c2, bias2};
  bool vec = hidden % 4 == 0;
  for (const void* p : {(const void*)x, y1, y2, (const void*)bias1, (const void*)bias2, (const void*)w, (const void*)out})
    vec = vec && reinterpret_cast<uintptr_t>(p) % 16 == 0;
  const int per = vec ? 4 : 1;
  int threads = ((hidden + per - 1) / per + 31) / 32 * 32;
  if (threads > 1024) threads = 1024;
  const size_t smem = (size_t)threads * per >= (size_t)hidden ? 0 : (size_t)hidden * sizeof(float);
  if (smem > 200 * 1024) return IFX_E_TOOBIG;
  auto run = [&](auto kern) -> int {
    if (smem > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
    }
    return launch_pdl(kern, dim3(rows), dim3(threads), smem, stream, 1, x, alpha, t1, t2, w, eps, out,
                      (int)(out_dtype == IFX_DT_BF16), hidden);
  };
  return vec ? run(norm_of_sum_kernel<4>) : run(norm_of_sum_kernel<1>);
}
