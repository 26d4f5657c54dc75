// Rotations of projected rows that need more than one head at a time, or the rows themselves back.
//
//   row_norm_rope_append   rows [nq heads of d | nkv key heads of d | nkv value heads of dv] (+ bias):
//                            queries: n_q(all of them together) * weight, turned, times a factor per head -> q_out
//                            keys:    n_k(all of them together) * weight, turned                          -> cache
//                            values:  turned by their own position over the whole head (optional)       -> cache
//                          With v_from_k there are no value columns: the values are the keys as projected (with their bias,
//                          in front of norm and rotation).  With gate_out: sigmoid of nq more columns, in float32.
//                          and the cosines and sines of the values' angles, for whoever turns a sum of values back.
//                          One block, or a cluster of blocks that share the heads, per token.
//   rotate_rows            rows [heads of d | heads of d | rest] -> float32: both groups of heads turned, the second one
//                          scaled behind it, the rest as it is.
//   silu_columns           rows -> float32, z / (1 + e^-z) on the first columns, the rest as it is.
//
// All read plain rows (wider ones than needed, from a column on) or the float32 partial sums of a K-split product.
// Angles are position * frequency in float32 with precise sines; norms, rotations and factors are float32.
#include <cooperative_groups.h>

#include "common.cuh"

namespace cg = cooperative_groups;

namespace ifx {

struct RowSource {
  const void* rows;            // plain rows, float32 or bfloat16, or null
  int is_bf16;
  const float* partial;        // partial sums [splits, tokens, ld], or null
  int splits;
  size_t split_stride;
  size_t ld;                   // elements from one token's row to the next
  int col0;                    // first column read

  __device__ __forceinline__ float2 load2(size_t token, int c) const {        // columns c and c + 1, c even
    const size_t at = token * ld + col0 + c;
    if (partial == nullptr) {
      if (is_bf16) return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(static_cast<const __nv_bfloat16*>(rows) + at));
      return *reinterpret_cast<const float2*>(static_cast<const float*>(rows) + at);
    }
    float2 s = make_float2(0.0f, 0.0f);
    for (int k = 0; k < splits; k += 4) {                    // four slices in flight, added in split order
      float2 part[4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        part[j] = k + j < splits ? *reinterpret_cast<const float2*>(partial + (size_t)(k + j) * split_stride + at) : make_float2(0.0f, 0.0f);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        s.x += part[j].x;
        s.y += part[j].y;
      }
    }
    return s;
  }
  __device__ __forceinline__ float load_one(size_t token, int c) const {
    if (partial == nullptr && is_bf16) return __bfloat162float(static_cast<const __nv_bfloat16*>(rows)[token * ld + col0 + c]);
    return partial == nullptr ? load1<false>(token, c) : load1<true>(token, c);
  }
  // float32 only; SLICED false (plain rows): a caller's loads are one straight run without a branch between them
  template <bool SLICED>
  __device__ __forceinline__ float load1(size_t token, int c) const {
    const size_t at = token * ld + col0 + c;
    if (!SLICED) return static_cast<const float*>(rows)[at];
    float s = 0.0f;
    for (int k = 0; k < splits; k += 4) {                    // four slices in flight, added in split order
      float part[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) part[j] = k + j < splits ? partial[(size_t)(k + j) * split_stride + at] : 0.0f;
#pragma unroll
      for (int j = 0; j < 4; ++j) s += part[j];
    }
    return s;
  }
};

struct RowRopeArgs {
  RowSource src;
  const float* bias;                           // [all columns] or null
  const float* q_norm; const float* k_norm;    // [nq d], [nkv d] or null
  float eps;
  const float* inv_freq; int rot, interleaved;            // queries and keys; rot 0: not turned
  const float* v_inv_freq; int v_interleaved;             // values, over all dv; null: not turned
  const float* temp;                           // [nq] or null
  const int* positions; const int* token_req; const int* req_slot; const int* block_table;
  int max_blocks, page_size, num_pages;
  void* kv_pool; void* q_out; float2* turn_out;
  int nq, nkv, d, dv, d_row, write_cache;
  int v_from_k;                                // value head g is read from key head g's columns
  float* gate_out; int gate_col;               // [tokens, nq] = sigmoid of the columns from gate_col on; null: no gate

  __device__ __forceinline__ int column(int u) const {        // the first column of unit u: queries, keys, values
    if (u < nq + nkv) return u * d;
    return v_from_k ? (u - nkv) * d : (nq + nkv) * d + (u - nq - nkv) * dv;
  }
  __device__ __forceinline__ void store_gate(int t) const {   // by all threads of a block
    if (gate_out == nullptr) return;
    for (int h = threadIdx.x; h < nq; h += blockDim.x) gate_out[(size_t)t * nq + h] = 1.0f / (1.0f + expf(-src.load_one(t, gate_col + h)));
  }
};

// element indices of pair j among a head's `size` elements of which `rot` turn
__device__ __forceinline__ void pair_of(int j, int rot, int interleaved, int& e0, int& e1) {
  const int half = rot / 2;
  if (j < half) {
    e0 = interleaved ? 2 * j : j;
    e1 = interleaved ? 2 * j + 1 : j + half;
  } else {
    e0 = rot + 2 * (j - half);
    e1 = e0 + 1;
  }
}

template <typename T>
__global__ void __launch_bounds__(1024) row_norm_rope_append_kernel(const RowRopeArgs a) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float part_q[32], part_k[32];
  __shared__ float total[2];
  const int t = blockIdx.x, z = blockIdx.z, C = gridDim.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
  const int units = a.nq + 2 * a.nkv, dmax = a.d > a.dv ? a.d : a.dv;
  const int half_rot = a.rot / 2, half_v = a.v_inv_freq ? a.dv / 2 : 0;
  float2* cs = reinterpret_cast<float2*>(smem);              // [half_rot] then [half_v]: (cos, sin)
  float* heads = smem + 2 * (half_rot + half_v);             // this block's heads, dmax apart
  pdl_launch_dependents();
  const int pos = a.positions[t];
  for (int j = threadIdx.x; j < half_rot + half_v; j += blockDim.x) {
    float sn, c;
    sincosf((float)pos * (j < half_rot ? a.inv_freq[j] : a.v_inv_freq[j - half_rot]), &sn, &c);
    cs[j] = make_float2(c, sn);
  }
  int page = -1;
  if (a.write_cache) page = a.block_table[(size_t)a.req_slot[a.token_req[t]] * a.max_blocks + pos / a.page_size];
  const bool page_ok = page >= 0 && page < a.num_pages;      // never write outside the pool
  pdl_wait();
  if (z == 0 && a.turn_out)
    for (int j = threadIdx.x; j < half_rot + half_v; j += blockDim.x)
      if (j >= half_rot) a.turn_out[(size_t)t * half_v + (j - half_rot)] = cs[j];      // this thread's own
  if (z == C - 1) a.store_gate(t);

  // ---- the rows, with their biases, and the sums of squares of all queries and of all keys
  float ss_q = 0.0f, ss_k = 0.0f;
  for (int u = z + warp * C, l = warp; u < units; u += nwarps * C, l += nwarps) {
    const bool is_v = u >= a.nq + a.nkv;
    const int size = is_v ? a.dv : a.d;
    const int col = a.column(u);
    float ss = 0.0f;
    for (int e = 2 * lane; e < size; e += 64) {
      float2 v = a.src.load2(t, col + e);
      if (a.bias) {
        v.x += a.bias[col + e];
        v.y += a.bias[col + e + 1];
      }
      ss = fmaf(v.x, v.x, ss);
      ss = fmaf(v.y, v.y, ss);
      *reinterpret_cast<float2*>(heads + (size_t)l * dmax + e) = v;
    }
    if (u < a.nq) ss_q += ss;
    else if (!is_v) ss_k += ss;
  }
  float inv_q = 1.0f, inv_k = 1.0f;
  if (a.q_norm != nullptr || a.k_norm != nullptr) {
    ss_q = warp_sum(ss_q);
    ss_k = warp_sum(ss_k);
    if (lane == 0) {
      part_q[warp] = ss_q;
      part_k[warp] = ss_k;
    }
    __syncthreads();
    ss_q = warp_sum(lane < nwarps ? part_q[lane] : 0.0f);
    ss_k = warp_sum(lane < nwarps ? part_k[lane] : 0.0f);
    if (C > 1) {
      if (threadIdx.x == 0) {
        total[0] = ss_q;
        total[1] = ss_k;
      }
      cg::cluster_group cluster = cg::this_cluster();
      cluster.sync();
      ss_q = ss_k = 0.0f;
      for (int b = 0; b < C; ++b) {                          // in block order: every block gets the same sum
        const float* other = cluster.map_shared_rank(total, b);
        ss_q += other[0];
        ss_k += other[1];
      }
      cluster.sync();                                        // nobody leaves while its sums are being read
    }
    inv_q = 1.0f / sqrtf(ss_q / (float)(a.nq * a.d) + a.eps);
    inv_k = 1.0f / sqrtf(ss_k / (float)(a.nkv * a.d) + a.eps);
  } else {
    __syncthreads();                                         // the angles
  }

  // ---- turned and stored, by the warp that loaded the head
  for (int u = z + warp * C, l = warp; u < units; u += nwarps * C, l += nwarps) {
    const bool is_q = u < a.nq, is_v = u >= a.nq + a.nkv;
    const int size = is_v ? a.dv : a.d;
    T* dst;
    if (is_q) {
      dst = static_cast<T*>(a.q_out) + ((size_t)t * a.nq + u) * a.d;
    } else {
      if (!page_ok) continue;
      const int g = u - a.nq - (is_v ? a.nkv : 0);
      dst = static_cast<T*>(a.kv_pool) +
            ((((size_t)page * 2 + (is_v ? 1 : 0)) * a.nkv + g) * a.page_size + (pos % a.page_size)) * a.d_row;
    }
    const float* hs = heads + (size_t)l * dmax;
    const float* nw = is_q ? a.q_norm : (is_v ? nullptr : a.k_norm);
    if (nw) nw += (size_t)(is_q ? u : u - a.nq) * a.d;
    const float inv = is_q ? inv_q : inv_k;
    const float factor = (is_q && a.temp) ? a.temp[u] : 1.0f;
    const int rot = is_v ? 2 * half_v : a.rot, half = rot / 2;
    const int inter = is_v ? a.v_interleaved : a.interleaved;
    const float2* angles = is_v ? cs + half_rot : cs;
    for (int j = lane; j < size / 2; j += 32) {
      int e0, e1;
      pair_of(j, rot, inter, e0, e1);
      float x = hs[e0], y = hs[e1];
      if (nw) {
        x = x * inv * nw[e0];
        y = y * inv * nw[e1];
      }
      if (j < half) {
        const float2 c = angles[j];
        const float rx = x * c.x - y * c.y, ry = y * c.x + x * c.y;
        x = rx;
        y = ry;
      }
      x *= factor;
      y *= factor;
      if (!is_q) {                                           // the cache only ever holds finite values
        x = isfinite(x) ? x : 0.0f;
        y = isfinite(y) ? y : 0.0f;
      }
      dst[e0] = from_f32<T>(x);
      dst[e1] = from_f32<T>(y);
    }
  }
}

// The same work for many tokens in the common case: plain bfloat16 rows, heads turned in halves, sizes and turned parts that
// are multiples of 4, up to 128.  A lane holds two pairs of every head of its warp: elements (2l, 2l + 1) and their partners
// half the turned part away, or, behind the turned part, the four elements from 4l on; all UPW heads in registers, fetched
// before anything is waited for.
template <int UPW>
__global__ void __launch_bounds__(512) row_norm_rope_rows_kernel(const RowRopeArgs a) {
  __shared__ __align__(16) float2 cs[128];                                 // [d / 2] then [dv / 2]
  __shared__ float part_q[16], part_k[16];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
  const int units = a.nq + 2 * a.nkv;
  const int half_rot = a.rot / 2, half_v = a.v_inv_freq ? a.dv / 2 : 0;
  const __nv_bfloat16* row = static_cast<const __nv_bfloat16*>(a.src.rows) + (size_t)t * a.src.ld + a.src.col0;
  const int pos = a.positions[t];
  int page = -1;
  if (a.write_cache) page = a.block_table[(size_t)a.req_slot[a.token_req[t]] * a.max_blocks + pos / a.page_size];
  pdl_wait();
  __nv_bfloat162 lo_raw[UPW], hi_raw[UPW];
  float2 lo[UPW], hi[UPW];
#pragma unroll
  for (int k = 0; k < UPW; ++k) {
    const int u = warp + k * nwarps;
    const bool is_v = u >= a.nq + a.nkv;
    const int half = (is_v ? a.dv : a.d) / 2, turned = is_v ? half_v : half_rot;
    const int e_lo = 2 * lane < turned ? 2 * lane : 4 * lane, e_hi = 2 * lane < turned ? 2 * lane + turned : 4 * lane + 2;
    const int col = a.column(u);
    lo_raw[k] = hi_raw[k] = __floats2bfloat162_rn(0.0f, 0.0f);
    lo[k] = hi[k] = make_float2(0.0f, 0.0f);
    if (u < units && 2 * lane < half) {
      lo_raw[k] = *reinterpret_cast<const __nv_bfloat162*>(row + col + e_lo);
      hi_raw[k] = *reinterpret_cast<const __nv_bfloat162*>(row + col + e_hi);
      if (a.bias) {
        lo[k] = *reinterpret_cast<const float2*>(a.bias + col + e_lo);
        hi[k] = *reinterpret_cast<const float2*>(a.bias + col + e_hi);
      }
    }
  }
  for (int j = threadIdx.x; j < half_rot + half_v; j += blockDim.x) {
    float sn, c;
    sincosf((float)pos * (j < half_rot ? a.inv_freq[j] : a.v_inv_freq[j - half_rot]), &sn, &c);
    cs[j] = make_float2(c, sn);
    if (j >= half_rot && a.turn_out) a.turn_out[(size_t)t * half_v + (j - half_rot)] = make_float2(c, sn);
  }
  a.store_gate(t);
  float ss_q = 0.0f, ss_k = 0.0f;
#pragma unroll
  for (int k = 0; k < UPW; ++k) {
    const int u = warp + k * nwarps;
    const float2 l = __bfloat1622float2(lo_raw[k]), h = __bfloat1622float2(hi_raw[k]);
    lo[k].x += l.x; lo[k].y += l.y; hi[k].x += h.x; hi[k].y += h.y;
    const float ss = fmaf(lo[k].x, lo[k].x, fmaf(lo[k].y, lo[k].y, fmaf(hi[k].x, hi[k].x, hi[k].y * hi[k].y)));
    if (u < a.nq) ss_q += ss;
    else if (u < a.nq + a.nkv) ss_k += ss;
  }
  ss_q = warp_sum(ss_q);
  ss_k = warp_sum(ss_k);
  if (lane == 0) {
    part_q[warp] = ss_q;
    part_k[warp] = ss_k;
  }
  __syncthreads();
  ss_q = warp_sum(lane < nwarps ? part_q[lane] : 0.0f);
  ss_k = warp_sum(lane < nwarps ? part_k[lane] : 0.0f);
  const float inv_q = 1.0f / sqrtf(ss_q / (float)(a.nq * a.d) + a.eps), inv_k = 1.0f / sqrtf(ss_k / (float)(a.nkv * a.d) + a.eps);
#pragma unroll
  for (int k = 0; k < UPW; ++k) {
    const int u = warp + k * nwarps;
    const bool is_q = u < a.nq, is_v = u >= a.nq + a.nkv;
    const int half = (is_v ? a.dv : a.d) / 2, turned = is_v ? half_v : half_rot;
    const int e_lo = 2 * lane < turned ? 2 * lane : 4 * lane, e_hi = 2 * lane < turned ? 2 * lane + turned : 4 * lane + 2;
    if (u >= units || 2 * lane >= half) continue;
    __nv_bfloat16* dst;
    if (is_q) {
      dst = static_cast<__nv_bfloat16*>(a.q_out) + ((size_t)t * a.nq + u) * a.d;
    } else {
      if (page < 0 || page >= a.num_pages) continue;         // never write outside the pool
      const int g = u - a.nq - (is_v ? a.nkv : 0);
      dst = static_cast<__nv_bfloat16*>(a.kv_pool) +
            ((((size_t)page * 2 + (is_v ? 1 : 0)) * a.nkv + g) * a.page_size + (pos % a.page_size)) * a.d_row;
    }
    float2 x = lo[k], y = hi[k];
    const float* nw = is_q ? a.q_norm : (is_v ? nullptr : a.k_norm);
    if (nw) {
      const float inv = is_q ? inv_q : inv_k;
      nw += (size_t)(is_q ? u : u - a.nq) * a.d;
      const float2 wl = *reinterpret_cast<const float2*>(nw + e_lo), wh = *reinterpret_cast<const float2*>(nw + e_hi);
      x.x *= inv * wl.x; x.y *= inv * wl.y; y.x *= inv * wh.x; y.y *= inv * wh.y;
    }
    if (2 * lane < turned) {
      const float4 c = *reinterpret_cast<const float4*>(&cs[(is_v ? half_rot : 0) + 2 * lane]);      // cos, sin of two pairs
      const float2 rx = make_float2(x.x * c.x - y.x * c.y, x.y * c.z - y.y * c.w);
      y = make_float2(y.x * c.x + x.x * c.y, y.y * c.z + x.y * c.w);
      x = rx;
    }
    if (is_q) {
      const float f = a.temp ? a.temp[u] : 1.0f;
      x.x *= f; x.y *= f; y.x *= f; y.y *= f;
    } else {                                                 // the cache only ever holds finite values
      x.x = isfinite(x.x) ? x.x : 0.0f;
      x.y = isfinite(x.y) ? x.y : 0.0f;
      y.x = isfinite(y.x) ? y.x : 0.0f;
      y.y = isfinite(y.y) ? y.y : 0.0f;
    }
    *reinterpret_cast<__nv_bfloat162*>(dst + e_lo) = __floats2bfloat162_rn(x.x, x.y);
    *reinterpret_cast<__nv_bfloat162*>(dst + e_hi) = __floats2bfloat162_rn(y.x, y.y);
  }
}

// A warp goes over the heads u, u + step, ... of one token: its lanes' angles are the same for all of them.  Four heads'
// elements are fetched before the first is stored (the rows may be turned where they lie).
template <bool SLICED>
__global__ void __launch_bounds__(128) rotate_rows_kernel(const RowSource src, const float* __restrict__ inv_freq, int rot,
                                                          int interleaved, const int* __restrict__ positions,
                                                          float* __restrict__ out, int width, int heads, int d, float k_scale,
                                                          int in_place) {
  pdl_launch_dependents();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int u0 = blockIdx.y * 4 + warp, step = gridDim.y * 4;
  const float pos = (float)positions[t];
  float* o = out + (size_t)t * width;
  bool arrived = false;
  for (int j = lane; j - lane < (d + 1) / 2; j += 32) {       // whole warps: a lane beyond the head does nothing
    const bool live = j < (d + 1) / 2;
    int e0, e1;
    pair_of(live ? j : 0, rot, interleaved, e0, e1);
    const bool both = e1 < d, turns = live && j < rot / 2;
    float2 c = make_float2(1.0f, 0.0f);
    if (turns) sincosf(pos * inv_freq[j], &c.y, &c.x);
    if (!arrived) pdl_wait();                                // angles do not come from the kernel in front
    arrived = true;
    for (int u = u0; u < 2 * heads; u += 4 * step) {
      float x[4], y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int h = u + k * step;
        const bool in = live && h < 2 * heads;
        x[k] = in ? src.load1<SLICED>(t, h * d + e0) : 0.0f;
        y[k] = in && both ? src.load1<SLICED>(t, h * d + e1) : 0.0f;
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int h = u + k * step;
        if (!live || h >= 2 * heads) continue;
        const float scale = h >= heads ? k_scale : 1.0f;
        const float rx = turns ? x[k] * c.x - y[k] * c.y : x[k], ry = turns ? y[k] * c.x + x[k] * c.y : y[k];
        o[h * d + e0] = rx * scale;
        if (both) o[h * d + e1] = ry * scale;
      }
    }
  }
  if (!arrived) pdl_wait();
  if (in_place) return;
  for (int c0 = 2 * heads * d + u0 * 128; c0 < width; c0 += step * 128)
    for (int c = c0 + lane; c < min(c0 + 128, width); c += 32) o[c] = src.load1<SLICED>(t, c);
}

// A warp takes 128 columns of one token at a time, four a lane.  `acted` columns get the activation; in place, only they
// are touched.
template <bool SLICED>
__global__ void __launch_bounds__(128) silu_columns_kernel(const RowSource src, float* __restrict__ out, int width, int acted,
                                                           int in_place) {
  pdl_launch_dependents();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int stop = in_place ? acted : width;
  float* o = out + (size_t)t * width;
  pdl_wait();
  for (int c0 = (blockIdx.y * 4 + warp) * 128 + lane; c0 - lane < stop; c0 += gridDim.y * 512) {
    float v[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) v[k] = c0 + 32 * k < stop ? src.load1<SLICED>(t, c0 + 32 * k) : 0.0f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int c = c0 + 32 * k;
      if (c < stop) o[c] = c < acted ? v[k] / (1.0f + expf(-v[k])) : v[k];
    }
  }
}

static int make_source(RowSource* s, const void* rows, int dtype, const float* partial, int splits, int tokens, long long ld, int col0) {
  if ((rows == nullptr) == (partial == nullptr) || ld <= 0 || col0 < 0) return IFX_E_BADARG;
  if (partial != nullptr && splits < 1) return IFX_E_BADARG;
  if (rows != nullptr && dtype != IFX_DT_F32 && dtype != IFX_DT_BF16) return IFX_E_DTYPE;
  *s = RowSource{rows, dtype == IFX_DT_BF16, partial, splits, (size_t)tokens * (size_t)ld, (size_t)ld, col0};
  return 0;
}

}  // namespace ifx

using namespace ifx;

extern "C" {

// Rows: `rows` (dtype src_dtype) or `partial` [splits, num_tokens, ld]; columns col0 .. col0 + (nq + nkv) d + nkv dv are read.
// turn_out: float2 [num_tokens, dv / 2] when v_inv_freq is given.  dtype: of q_out and the cache.
// v_from_k: columns col0 .. col0 + (nq + nkv) d are read, bias has that size, dv == d.
// gate_out: null, or float32 [num_tokens, nq]; its columns begin at col0 + gate_col.
int ifx_row_norm_rope_append(const void* rows, int src_dtype, const float* partial, int splits, long long ld, int col0,
                             const float* bias, const float* q_norm, const float* k_norm, float eps, const float* inv_freq,
                             int rot, int interleaved, const float* v_inv_freq, int v_interleaved, const float* temp,
                             const int* positions, const int* token_req, const int* req_slot, const int* block_table,
                             int max_blocks, int page_size, int num_pages, void* kv_pool, void* q_out, float* turn_out,
                             int num_tokens, int nq, int nkv, int d, int dv, int d_row, int write_cache, int v_from_k,
                             float* gate_out, int gate_col, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || nq % nkv || d <= 0 || d % 2 || dv <= 0 || dv % 2 || rot < 0 || rot > d || rot % 2 || ld % 2 || col0 % 2 ||
      (rot > 0 && inv_freq == nullptr) || q_out == nullptr)
    return IFX_E_BADARG;
  if (col0 + (long long)(nq + nkv) * d + (v_from_k ? 0 : (long long)nkv * dv) > ld || (v_from_k && dv != d)) return IFX_E_BADARG;
  if (gate_out != nullptr && (gate_col < 0 || (long long)col0 + gate_col + nq > ld)) return IFX_E_BADARG;
  if (write_cache && (page_size <= 0 || max_blocks <= 0 || kv_pool == nullptr || block_table == nullptr || d_row < d || d_row < dv))
    return IFX_E_BADARG;
  if (dtype != IFX_DT_F32 && dtype != IFX_DT_BF16) return IFX_E_DTYPE;
  RowRopeArgs a{};
  const int rc = make_source(&a.src, rows, src_dtype, partial, splits, num_tokens, ld, col0);
  if (rc) return rc;
  for (const void* p : {rows, (const void*)partial})
    if (reinterpret_cast<uintptr_t>(p) % 8) return IFX_E_ALIGN;
  a.bias = bias; a.q_norm = q_norm; a.k_norm = k_norm; a.eps = eps; a.inv_freq = inv_freq; a.rot = rot; a.interleaved = interleaved;
  a.v_inv_freq = v_inv_freq; a.v_interleaved = v_interleaved; a.temp = temp; a.positions = positions; a.token_req = token_req;
  a.req_slot = req_slot; a.block_table = block_table; a.max_blocks = max_blocks; a.page_size = page_size; a.num_pages = num_pages;
  a.kv_pool = kv_pool; a.q_out = q_out; a.turn_out = reinterpret_cast<float2*>(turn_out); a.nq = nq; a.nkv = nkv; a.d = d; a.dv = dv;
  a.d_row = d_row; a.write_cache = write_cache; a.v_from_k = v_from_k; a.gate_out = gate_out; a.gate_col = gate_col;
  const int units = nq + 2 * nkv, dmax = d > dv ? d : dv;
  auto aligned = [](const void* p, int n) { return reinterpret_cast<uintptr_t>(p) % n == 0; };
  if (dtype == IFX_DT_BF16 && rows != nullptr && src_dtype == IFX_DT_BF16 && num_tokens > 32 && rot % 4 == 0 && !interleaved &&
      (v_inv_freq == nullptr || !v_interleaved) && d % 4 == 0 && dv % 4 == 0 && dmax <= 128 && units <= 64 && d_row % 2 == 0 &&
      aligned(bias, 8) && aligned(q_norm, 8) && aligned(k_norm, 8) && aligned(q_out, 4) && aligned(kv_pool, 4)) {
    const int per_warp = (units + 15) / 16, warps = (units + per_warp - 1) / per_warp;
    const dim3 grid(num_tokens), block(32 * warps);
    switch (per_warp) {
      case 1: return launch_pdl(row_norm_rope_rows_kernel<1>, grid, block, 0, stream, 1, a);
      case 2: return launch_pdl(row_norm_rope_rows_kernel<2>, grid, block, 0, stream, 1, a);
      case 3: return launch_pdl(row_norm_rope_rows_kernel<3>, grid, block, 0, stream, 1, a);
      default: return launch_pdl(row_norm_rope_rows_kernel<4>, grid, block, 0, stream, 1, a);
    }
  }
  // Few bfloat16 tokens: a cluster of blocks shares a token's heads, so that more than one SM fetches its slices.  Float32
  // runs keep one block a token, so that the order of a row's additions never depends on the step.
  int C = 1;
  if (dtype == IFX_DT_BF16 && num_tokens <= 32 && units >= 16) C = num_tokens <= 16 ? 8 : 4;
  const int local = (units + C - 1) / C;
  const int threads = 32 * (local < 16 ? local : 16);
  const size_t smem = ((size_t)local * dmax + rot + (v_inv_freq ? dv : 0)) * sizeof(float);
  if (smem > 220 * 1024) return IFX_E_TOOBIG;
  auto run = [&](auto kern) -> int {
    if (smem > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
    }
    return launch_pdl(kern, dim3(num_tokens, 1, C), dim3(threads), smem, stream, C, a);
  };
  return dtype == IFX_DT_F32 ? run(row_norm_rope_append_kernel<float>) : run(row_norm_rope_append_kernel<__nv_bfloat16>);
}

// float32 rows in (plain or partial sums), float32 [num_tokens, width] out; out may be `rows` itself when ld == width and
// col0 == 0 (in_place: the rest is then left alone).
int ifx_rotate_rows(const float* rows, const float* partial, int splits, long long ld, int col0, const float* inv_freq, int rot,
                    int interleaved, const int* positions, float* out, int num_tokens, int width, int heads, int d, float k_scale,
                    cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (heads <= 0 || d <= 0 || rot < 0 || rot > d || rot % 2 || width < 2 * heads * d || col0 + (long long)width > ld ||
      (rot > 0 && inv_freq == nullptr) || out == nullptr)
    return IFX_E_BADARG;
  const int in_place = rows == out;
  if (in_place && (ld != width || col0 != 0)) return IFX_E_BADARG;
  RowSource src;
  const int rc = make_source(&src, rows, IFX_DT_F32, partial, splits, num_tokens, ld, col0);
  if (rc) return rc;
  // few tokens: a head (or 128 columns of the rest) a warp; many: one block a token
  const int rest = in_place ? 0 : (width - 2 * heads * d + 127) / 128, most = 2 * heads > rest ? 2 * heads : rest;
  int blocks = num_tokens >= 128 ? 1 : (most + 3) / 4;
  if (blocks > 1024) blocks = 1024;
  return launch_pdl(partial ? rotate_rows_kernel<true> : rotate_rows_kernel<false>, dim3(num_tokens, blocks), dim3(128), 0, stream, 1, src, inv_freq, rot, interleaved,
                    positions, out, width, heads, d, k_scale, in_place);
}

// float32 rows in (plain or partial sums), float32 [num_tokens, width] out: silu on the first `acted` columns, the others as
// they are; out may be `rows` itself when ld == width and col0 == 0.
int ifx_silu_columns(const float* rows, const float* partial, int splits, long long ld, int col0, float* out, int num_tokens,
                     int width, int acted, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (width <= 0 || acted < 0 || acted > width || col0 + (long long)width > ld || out == nullptr) return IFX_E_BADARG;
  const int in_place = rows == out;
  if (in_place && (ld != width || col0 != 0)) return IFX_E_BADARG;
  RowSource src;
  const int rc = make_source(&src, rows, IFX_DT_F32, partial, splits, num_tokens, ld, col0);
  if (rc) return rc;
  int blocks = ((in_place ? acted : width) + 511) / 512;
  if (blocks < 1) blocks = 1;
  if (blocks > 1024) blocks = 1024;
  return launch_pdl(partial ? silu_columns_kernel<true> : silu_columns_kernel<false>, dim3(num_tokens, blocks), dim3(128), 0, stream, 1, src,
                    out, width, acted, in_place);
}

}  // extern "C"
