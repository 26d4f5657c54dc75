// An elementwise recurrence whose gates read the present token only:
//
//   z = sigmoid(zr + bz),  u = ur + bu,  c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0)
//   S <- (1 - z) S + z c,  out = S * silu(g)                  S: one float32 number per request and channel
//
// rows [T, 3 width] hold zr, ur, g side by side in float32, plain or as the partial sums [splits, T, 3 width] of a
// K-split product.  state: a slot per request, slot_stride floats apart; a new request finds it zeroed.
//
// A span of many tokens is walked in tiles of 64 tokens x 32 channels.  Only the multiply-add S <- a S + b has to go from
// token to token: one warp does that, a channel a lane, out of shared memory, while the other warps turn the next tile's
// projections (fetched into registers a tile ahead) into its a and b and the tile before into output.  Every S is the
// same chain of multiply-adds however the tokens are cut into steps.
#include "common.cuh"

namespace ifx {

struct GatedScanArgs {
  const float* rows; int splits; size_t split_stride;
  const float* bias;                            // [2 width]
  float* state; long long slot_stride;
  const int* req_slot; const int* cu_seqlens;
  void* out;
  int width;
};

// sigmoid(|v|) and sigmoid(-|v|); the divisor lies between 1 and 2, where the fast division is good to an ulp or two
__device__ __forceinline__ void sigmoid_pair(float v, float& big, float& small) {
  const float e = expf(-fabsf(v));
  big = __fdividef(1.0f, 1.0f + e);
  small = e * big;
}
__device__ __forceinline__ float sigmoid_f32(float v) {
  float big, small;
  sigmoid_pair(v, big, small);
  return v >= 0.0f ? big : small;
}

// SLICED false: plain rows, so that a caller's loads are one straight run without a loop between them.
template <bool SLICED>
__device__ __forceinline__ float load_sliced(const GatedScanArgs& a, size_t at) {
  float s = __ldcg(a.rows + at);
  if constexpr (SLICED) {
    for (int k = 1; k < a.splits; k += 4) {                   // four slices in flight, added in split order
      float part[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) part[j] = k + j < a.splits ? __ldcg(a.rows + (size_t)(k + j) * a.split_stride + at) : 0.0f;
#pragma unroll
      for (int j = 0; j < 4; ++j) s += part[j];
    }
  }
  return s;
}

// what a token does to S: S <- keep S + take
__device__ __forceinline__ void gate_of(float zr, float u, float& keep, float& take) {
  float big, small;
  sigmoid_pair(zr, big, small);
  keep = zr >= 0.0f ? small : big;
  take = (zr >= 0.0f ? big : small) * (u >= 0.0f ? u + 0.5f : sigmoid_f32(u));
}

// One token a request: a thread per channel.
template <typename T>
__global__ void __launch_bounds__(128) gated_step_kernel(const GatedScanArgs a) {
  pdl_launch_dependents();
  const int c = blockIdx.x * blockDim.x + threadIdx.x, r = blockIdx.y;
  const bool live = c < a.width;
  const size_t t = (size_t)a.cu_seqlens[r];
  const int slot = a.req_slot[r];
  const float bz = live ? a.bias[c] : 0.0f, bu = live ? a.bias[a.width + c] : 0.0f;
  pdl_wait();
  if (!live) return;
  float* st = a.state + (long long)slot * a.slot_stride + c;
  const float S0 = *st;
  const size_t at = t * 3 * a.width + c;
  const float zr = load_sliced<true>(a, at) + bz, u = load_sliced<true>(a, at + a.width) + bu;
  const float g = load_sliced<true>(a, at + 2 * (size_t)a.width);
  float keep, take;
  gate_of(zr, u, keep, take);
  const float S = fmaf(keep, S0, take);
  *st = S;
  static_cast<T*>(a.out)[t * a.width + c] = from_f32<T>(S * (g * sigmoid_f32(g)));
}

constexpr int kScanTokens = 64, kScanWorkers = 16, kScanPer = kScanTokens / kScanWorkers;     // tokens a worker warp holds

template <typename T, bool SLICED>
__global__ void __launch_bounds__((kScanWorkers + 1) * 32) gated_scan_kernel(const GatedScanArgs a) {
  __shared__ float keep_s[2][kScanTokens][32], take_s[2][kScanTokens][32];     // take becomes S as the walk passes
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * 32 + lane, r = blockIdx.y;
  const bool live = c < a.width;
  pdl_launch_dependents();
  const int first = a.cu_seqlens[r], n = a.cu_seqlens[r + 1] - first;
  const int tiles = (n + kScanTokens - 1) / kScanTokens;
  float* st = a.state + (long long)a.req_slot[r] * a.slot_stride + c;
  const float bz = live ? a.bias[c] : 0.0f, bu = live ? a.bias[a.width + c] : 0.0f;
  pdl_wait();
  if (warp == kScanWorkers) {                                // ---- the walk
    float S = live ? *st : 0.0f;
    __syncthreads();                                         // tile 0 is there
    for (int i = 0; i < tiles; ++i) {
      const int b = i & 1, m = min(kScanTokens, n - i * kScanTokens);
      int t = 0;
      for (; t + 16 <= m; t += 16) {
        float k[16], v[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          k[j] = keep_s[b][t + j][lane];
          v[j] = take_s[b][t + j][lane];
        }
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          S = fmaf(k[j], S, v[j]);
          take_s[b][t + j][lane] = S;
        }
      }
      for (; t < m; ++t) {
        S = fmaf(keep_s[b][t][lane], S, take_s[b][t][lane]);
        take_s[b][t][lane] = S;
      }
      __syncthreads();
    }
    if (live) *st = S;
    return;
  }
  // ---- the others: a warp owns tokens warp, warp + 16, ... of every tile
  float zr[kScanPer], ur[kScanPer], gr[kScanPer], gate[kScanPer];
  auto fetch = [&](int i) {
#pragma unroll
    for (int j = 0; j < kScanPer; ++j) {
      const int t = i * kScanTokens + warp + j * kScanWorkers;
      zr[j] = ur[j] = gr[j] = 0.0f;
      if (live && t < n) {
        const size_t at = (size_t)(first + t) * 3 * a.width + c;
        zr[j] = load_sliced<SLICED>(a, at);
        ur[j] = load_sliced<SLICED>(a, at + a.width);
        gr[j] = load_sliced<SLICED>(a, at + 2 * (size_t)a.width);
      }
    }
  };
  auto make = [&](int b) {
#pragma unroll
    for (int j = 0; j < kScanPer; ++j) {
      float keep, take;
      gate_of(zr[j] + bz, ur[j] + bu, keep, take);
      keep_s[b][warp + j * kScanWorkers][lane] = keep;
      take_s[b][warp + j * kScanWorkers][lane] = take;
    }
  };
  auto hold_gates = [&]() {
#pragma unroll
    for (int j = 0; j < kScanPer; ++j) gate[j] = gr[j] * sigmoid_f32(gr[j]);
  };
  float next_gate[kScanPer];
  fetch(0);
  make(0);
  hold_gates();
  fetch(1);
  __syncthreads();
  for (int i = 0; i < tiles; ++i) {
    if (i + 1 < tiles) {
      make((i + 1) & 1);                                     // its last readers were this warp's own lanes, a tile ago
#pragma unroll
      for (int j = 0; j < kScanPer; ++j) next_gate[j] = gr[j] * sigmoid_f32(gr[j]);
      fetch(i + 2);
    }
    __syncthreads();                                         // tile i has been walked, tile i + 1 is there
#pragma unroll
    for (int j = 0; j < kScanPer; ++j) {
      const int t = i * kScanTokens + warp + j * kScanWorkers;
      if (live && t < n)
        static_cast<T*>(a.out)[(size_t)(first + t) * a.width + c] = from_f32<T>(take_s[i & 1][warp + j * kScanWorkers][lane] * gate[j]);
      gate[j] = next_gate[j];
    }
  }
}

}  // namespace ifx

using namespace ifx;

// rows: float32 [splits, num_tokens, 3 width] (splits 1: plain).  max_span: the most tokens a request brings.
extern "C" int ifx_gated_scan(const float* rows, int splits, const float* bias, float* state, long long slot_stride,
                              const int* req_slot, const int* cu_seqlens, void* out, int num_requests, int num_tokens, int max_span,
                              int width, int out_dtype, cudaStream_t stream) {
  if (num_requests <= 0 || num_tokens <= 0) return 0;
  if (width <= 0 || splits < 1 || max_span <= 0 || slot_stride < width) return IFX_E_BADARG;
  if (num_requests > 65535) return IFX_E_TOOBIG;
  if (out_dtype != IFX_DT_F32 && out_dtype != IFX_DT_BF16) return IFX_E_DTYPE;
  GatedScanArgs a{rows, splits, (size_t)num_tokens * 3 * width, bias, state, slot_stride, req_slot, cu_seqlens, out, width};
  const bool f32 = out_dtype == IFX_DT_F32;
  if (max_span == 1) {
    const dim3 grid((width + 127) / 128, num_requests);
    return launch_pdl(f32 ? gated_step_kernel<float> : gated_step_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, 1, a);
  }
  const dim3 grid((width + 31) / 32, num_requests);
  const dim3 block((kScanWorkers + 1) * 32);
  if (splits > 1)
    return launch_pdl(f32 ? gated_scan_kernel<float, true> : gated_scan_kernel<__nv_bfloat16, true>, grid, block, 0, stream, 1, a);
  return launch_pdl(f32 ? gated_scan_kernel<float, false> : gated_scan_kernel<__nv_bfloat16, false>, grid, block, 0, stream, 1, a);
}
