// Shared helpers of the sm_100a kernels: dtype conversion, warp/block reductions,
// argument checks.  Every exported function returns 0 on success, a positive
// cudaError_t, or a negative IFX_E_* code for arguments it refuses.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define IFX_DT_F32 0
#define IFX_DT_BF16 1

#define IFX_E_BADARG (-1)      // a size or option the kernel does not take
#define IFX_E_DTYPE (-2)       // unknown dtype code
#define IFX_E_ALIGN (-3)       // a pointer or stride that breaks an alignment rule
#define IFX_E_TOOBIG (-4)      // beyond a stated maximum

#define IFX_CHECK_LAUNCH()                         \
  do {                                             \
    cudaError_t e__ = cudaGetLastError();          \
    if (e__ != cudaSuccess) return (int)e__;       \
  } while (0)

namespace ifx {

// Programmatic dependent launch: a kernel launched with launch_pdl may begin (set up
// its barriers, fetch weights) while the kernel before it in the stream is still
// draining; pdl_wait() returns once that kernel has completed and its writes are
// visible, and must come before the first access to anything it produced.  Every
// kernel launched this way calls pdl_wait() at some point, so completion stays
// transitive along the stream.  pdl_launch_dependents() lets the next kernel's
// blocks take the SM slots this kernel's blocks leave.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

extern int g_pdl_enabled;      // 1: launch_pdl sets the programmatic-serialization attribute
extern int g_shared_carveout;  // >= 0: percent of the SM's memory every launch_pdl kernel prefers as shared memory

template <typename... KArgs, typename... Args>
inline int launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                      int cluster_z, Args... args) {
  if (g_shared_carveout >= 0) {
    // Every kernel of the chain asks for the same split of the SM's memory into shared memory and L1, so that
    // no SM has to drain to change it between two kernels (measured: 3.30 -> 3.23 ms for a decode step of the
    // 7B shape at batch 8 with 100, 3.87 ms with 50).
    static const void* configured[64];                   // kernels of this signature seen so far
    static int num_configured = 0;
    const void* fn = reinterpret_cast<const void*>(kernel);
    bool seen = false;
    for (int i = 0; i < num_configured; ++i) seen = seen || configured[i] == fn;
    if (!seen) {
      cudaFuncSetAttribute(fn, cudaFuncAttributePreferredSharedMemoryCarveout, g_shared_carveout);
      if (num_configured < 64) configured[num_configured++] = fn;
    }
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (cluster_z > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = 1;
    attr[n].val.clusterDim.y = 1;
    attr[n].val.clusterDim.z = cluster_z;
    ++n;
  }
  if (g_pdl_enabled) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n;
  cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
  return e == cudaSuccess ? 0 : (int)e;
}

// Which keys a query sees besides "not later than itself": the last `window` of them (> 0), only those of its own
// stretch of `chunk` positions (> 0), or both; the first `keep` keys of a sequence stay visible whatever the window or the
// stretch.  A query's keys are therefore [0, kept(first)) and [first, pos].  `sink`: the softmax's denominator holds one more unit, a key of score 0
// that brings no value; with `sink_values` (one learned number per query head) the unit is exp(that number) instead.
struct KeyMask {
  int window, chunk, sink;
  const float* sink_values;
  int keep;
  // the sink's score in units of log2, for kernels that keep maxima and sums as powers of two
  __device__ __forceinline__ float sink_log2(int head) const {
    return sink_values ? sink_values[head] * 1.4426950408889634f : 0.0f;
  }
  __device__ __forceinline__ int first(int pos) const {          // the first key the query at `pos` sees
    int f = window > 0 ? max(0, pos - window + 1) : 0;
    if (chunk > 0) f = max(f, pos / chunk * chunk);
    return f;
  }
  __device__ __forceinline__ bool any() const { return window > 0 || chunk > 0; }
  __device__ __forceinline__ int kept(int first) const { return min(keep, first); }      // keys in front of `first` that stay
  __device__ __forceinline__ bool sees(int key, int first) const { return key >= first || key < keep; }
};

// What happens to a head's finished sum of values before it is rounded and stored.
// Values that were turned by their own position before they were summed: the sum is turned back by the query's.  `table`
// [tokens, size / 2] holds cos and sin of the query's angles (null: nothing is turned); pairs are (m, m + size / 2), or
// neighbours with `interleaved`.
// A gate per token and head: the sum is multiplied by gate[token, head] of `heads` a row (null: 1).
struct HeadOutput {
  const float2* table;
  int interleaved;
  const float* gate;
  int heads;
  __device__ __forceinline__ float factor(int token, int head) const {
    return gate ? gate[(size_t)token * heads + head] : 1.0f;
  }
  __device__ __forceinline__ static void apply(float2 cs, float& u, float& v) {
    const float a = u * cs.x + v * cs.y, b = v * cs.x - u * cs.y;
    u = a;
    v = b;
  }
};

// The tanh form of gelu, z/2 (1 + tanh(s (z + 0.044715 z^3))) with s = sqrt(2/pi), as z sigmoid(2 s (z + 0.044715 z^3)).
__device__ __forceinline__ float gelu_tanh_f32(float z) {
  const float u = 1.5957691216057308f * fmaf(0.044715f * z * z, z, z);
  return z / (1.0f + expf(-u));
}
// The same with the fast exponential and division: a few float32 ulps, for results that are rounded to bfloat16.
__device__ __forceinline__ float gelu_tanh_fast(float z) {
  const float u = 1.5957691216057308f * fmaf(0.044715f * z * z, z, z);
  return __fdividef(z, 1.0f + __expf(fminf(-u, 80.0f)));
}

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) {
  return __float2bfloat16_rn(v);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result.  The order
// of the additions depends only on the block size, so a row's result does not
// depend on which other rows are in the launch.
__device__ __forceinline__ float block_sum(float v, float* scratch /* >= 32 floats */) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();                       // scratch may still be read from a previous call
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float r = (lane < nwarps) ? scratch[lane] : 0.0f;
  r = warp_sum(r);
  return r;
}

__device__ __forceinline__ float block_max(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float r = (lane < nwarps) ? scratch[lane] : -INFINITY;
  r = warp_max(r);
  return r;
}

}  // namespace ifx
