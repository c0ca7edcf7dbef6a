// Routing of a drop-free mixture of experts: the `top` largest sigmoid scores of every token, rows sorted by
// expert and scaled by the score, and the sum over a token's choices afterwards.
//
//   route_small_kernel   few pairs: ONE launch.  Every CTA routes all tokens for itself (the logits are a few
//                        kilobytes), so that no CTA waits for another, and gathers its share of the rows.
//   route_topk / route_layout / route_gather   many pairs: scores and places, offsets, rows.
//   expert_combine_kernel   out[t] = sum over choices of y[place].
//
// A pair is token * top + choice.  Places inside an expert's run may differ from launch to launch in the
// three-kernel form; results do not depend on them.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "mma_sync.cuh"

namespace axb {

struct RouteArgs {
  const float* logits;   // [tokens, logits_ld]
  const void* h;         // [tokens, h_ld]
  int* ids;              // [pairs]
  float* weight;         // [pairs]
  int* place;            // [pairs] row of the pair
  int* offsets;          // [experts + 1] first row of every expert, runs rounded up to `block`
  int* block_expert;     // [blocks] owner of every block of rows, -1: none
  int* row_pair;         // [rows] pair of a row (block 1)
  void* rows_out;        // [rows, rows_ld]
  int* counts;           // [experts]
  int64_t logits_ld, h_ld, rows_ld;
  int tokens, experts, top, width, block, blocks, act_bf16;
};

namespace {

constexpr int kRtThreads = 256, kRtWarps = kRtThreads / 32, kRtMaxExperts = 1024, kRtMaxPairs = 1024;

__device__ __forceinline__ float rf(float x) { return x; }
__device__ __forceinline__ float rf(__nv_bfloat16 x) { return __bfloat162float(x); }

// The warp's lanes hold the logits of experts lane + 32 i; calls put(choice, expert, score) on every lane.
// Equal logits: the lower expert first.
template <int EPL, typename F>
__device__ __forceinline__ void warp_topk(const float* logits, int experts, int top, F put) {
  const int lane = threadIdx.x & 31;
  float v[EPL];
#pragma unroll
  for (int i = 0; i < EPL; ++i) v[i] = lane + 32 * i < experts ? logits[lane + 32 * i] : -INFINITY;
  uint32_t taken = 0;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < EPL; ++i)
      if (!(taken >> i & 1) && lane + 32 * i < experts && (at == 0x7fffffff || v[i] > best)) best = v[i], at = lane + 32 * i;
    for (int off = 16; off > 0; off >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, off);
      const int oa = __shfl_xor_sync(0xffffffffu, at, off);
      if (oa != 0x7fffffff && (at == 0x7fffffff || ov > best || (ov == best && oa < at))) best = ov, at = oa;
    }
    if ((at & 31) == lane) taken |= 1u << (at >> 5);
    put(k, at, 1.f / (1.f + expf(-best)));
  }
}

template <typename T>
__device__ __forceinline__ void scaled_row(const RouteArgs& a, int token, float w, int64_t row, int tid, int threads) {
  const T* src = static_cast<const T*>(a.h) + token * a.h_ld;
  T* dst = static_cast<T*>(a.rows_out) + row * a.rows_ld;
  if (sizeof(T) == 2 && !((a.h_ld | a.rows_ld | a.width) & 7)) {
    for (int c = tid * 8; c < a.rows_ld; c += threads * 8) {
      uint4 o = make_uint4(0, 0, 0, 0);
      if (c < a.width) {
        const uint4 u = *reinterpret_cast<const uint4*>(src + c);
        const uint32_t in[4] = {u.x, u.y, u.z, u.w};
        uint32_t r[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = unpack2(in[i]);
          r[i] = pack2(f.x * w, f.y * w);
        }
        o = make_uint4(r[0], r[1], r[2], r[3]);
      }
      *reinterpret_cast<uint4*>(dst + c) = o;
    }
  } else {
    for (int c = tid; c < a.rows_ld; c += threads) dst[c] = c < a.width ? T(rf(src[c]) * w) : T(0.f);
  }
}

}  // namespace

constexpr int kRsThreads = 512, kRsWarps = kRsThreads / 32;

template <typename T, int EPL>
__global__ void __launch_bounds__(kRsThreads) route_small_kernel(RouteArgs a) {
  __shared__ int s_id[kRtMaxPairs], s_place[kRtMaxPairs], s_base[kRtMaxExperts + 1];
  __shared__ float s_w[kRtMaxPairs];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, pairs = a.tokens * a.top;
  for (int t = warp; t < a.tokens; t += kRsWarps)
    warp_topk<EPL>(a.logits + t * a.logits_ld, a.experts, a.top, [&](int k, int e, float s) {
      if (lane == 0) s_id[t * a.top + k] = e, s_w[t * a.top + k] = s;
    });
  __syncthreads();
  for (int e = warp; e < a.experts; e += kRsWarps) {
    int run = 0;
    for (int p0 = 0; p0 < pairs; p0 += 32) {
      const bool mine = p0 + lane < pairs && s_id[p0 + lane] == e;
      const uint32_t mask = __ballot_sync(0xffffffffu, mine);
      if (mine) s_place[p0 + lane] = run + __popc(mask & ((1u << lane) - 1));
      run += __popc(mask);
    }
    if (lane == 0) s_base[e + 1] = run;
  }
  __syncthreads();
  if (warp == 0) {
    int carry = 0;
    if (lane == 0) s_base[0] = 0;
    for (int e0 = 0; e0 < a.experts; e0 += 32) {
      int x = e0 + lane < a.experts ? s_base[e0 + lane + 1] : 0;
      for (int off = 1; off < 32; off <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, x, off);
        if (lane >= off) x += y;
      }
      if (e0 + lane < a.experts) s_base[e0 + lane + 1] = carry + x;
      carry += __shfl_sync(0xffffffffu, x, 31);
    }
  }
  __syncthreads();
  if (blockIdx.x == 0) {
    for (int e = tid; e <= a.experts; e += kRsThreads) a.offsets[e] = s_base[e];
    for (int p = tid; p < pairs; p += kRsThreads) a.row_pair[s_base[s_id[p]] + s_place[p]] = p;
  }
  for (int p = blockIdx.x * 2 + (tid >> 8); p < pairs; p += gridDim.x * 2)
    scaled_row<T>(a, p / a.top, s_w[p], s_base[s_id[p]] + s_place[p], tid & 255, 256);
}

constexpr int kRtTokens = 64;  // tokens per CTA of the three-kernel form

// Places come from a count of the CTA's own pairs in shared memory and one addition per (CTA, expert) to the
// expert's total.
template <int EPL>
__global__ void __launch_bounds__(kRtThreads) route_topk_kernel(RouteArgs a) {
  extern __shared__ int s_count[];  // [experts]: pairs of this CTA, then their first place
  const int tid = threadIdx.x, lane = tid & 31, t0 = blockIdx.x * kRtTokens;
  const int t1 = min(a.tokens, t0 + kRtTokens);
  for (int e = tid; e < a.experts; e += kRtThreads) s_count[e] = 0;
  __syncthreads();
  for (int t = t0 + (tid >> 5); t < t1; t += kRtWarps)
    warp_topk<EPL>(a.logits + t * a.logits_ld, a.experts, a.top, [&](int k, int e, float s) {
      if (lane == 0) {
        const int p = t * a.top + k;
        a.ids[p] = e;
        a.weight[p] = s;
        a.place[p] = atomicAdd(s_count + e, 1);
      }
    });
  __syncthreads();
  for (int e = tid; e < a.experts; e += kRtThreads)
    if (s_count[e] > 0) s_count[e] = atomicAdd(a.counts + e, s_count[e]);
  __syncthreads();
  for (int p = t0 * a.top + tid; p < t1 * a.top; p += kRtThreads) a.place[p] += s_count[a.ids[p]];
}

// One CTA.
__global__ void __launch_bounds__(kRtThreads) route_layout_kernel(RouteArgs a) {
  __shared__ int s_base[kRtMaxExperts + 1];
  const int tid = threadIdx.x, lane = tid & 31;
  if (tid < 32) {
    int carry = 0;
    if (lane == 0) s_base[0] = 0;
    for (int e0 = 0; e0 < a.experts; e0 += 32) {
      int x = e0 + lane < a.experts ? (a.counts[e0 + lane] + a.block - 1) / a.block * a.block : 0;
      for (int off = 1; off < 32; off <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, x, off);
        if (lane >= off) x += y;
      }
      if (e0 + lane < a.experts) s_base[e0 + lane + 1] = carry + x;
      carry += __shfl_sync(0xffffffffu, x, 31);
    }
  }
  __syncthreads();
  for (int e = tid; e <= a.experts; e += kRtThreads) a.offsets[e] = s_base[e];
  if (a.block == 1) return;
  for (int i = tid; i < a.blocks; i += kRtThreads) {
    const int r = i * a.block;
    int lo = 0, hi = a.experts;  // the last expert whose run starts at or ahead of r
    while (hi - lo > 1) {
      const int mid = (lo + hi) / 2;
      if (s_base[mid] <= r) lo = mid;
      else hi = mid;
    }
    a.block_expert[i] = r < s_base[a.experts] ? lo : -1;
  }
}

// A token's row is read once and written `top` times.
template <typename T>
__global__ void __launch_bounds__(kRtThreads) route_gather_kernel(RouteArgs a) {
  extern __shared__ int s_row[];  // [top]
  const int t = blockIdx.x, tid = threadIdx.x;
  for (int k = tid; k < a.top; k += kRtThreads) {
    const int p = t * a.top + k, row = a.offsets[a.ids[p]] + a.place[p];
    s_row[k] = row;
    a.place[p] = row;
    if (a.block == 1) a.row_pair[row] = p;
  }
  __syncthreads();
  const T* src = static_cast<const T*>(a.h) + t * a.h_ld;
  T* out = static_cast<T*>(a.rows_out);
  const float* weight = a.weight + static_cast<int64_t>(t) * a.top;
  if (sizeof(T) == 2 && !((a.h_ld | a.rows_ld | a.width) & 7)) {
    for (int c = tid * 8; c < a.rows_ld; c += kRtThreads * 8) {
      float f[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = 0.f;
      if (c < a.width) {
        const uint4 u = *reinterpret_cast<const uint4*>(src + c);
        const uint32_t in[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 x = unpack2(in[i]);
          f[2 * i] = x.x, f[2 * i + 1] = x.y;
        }
      }
      for (int k = 0; k < a.top; ++k) {
        const float w = weight[k];
        *reinterpret_cast<uint4*>(out + s_row[k] * a.rows_ld + c) =
            make_uint4(pack2(f[0] * w, f[1] * w), pack2(f[2] * w, f[3] * w), pack2(f[4] * w, f[5] * w), pack2(f[6] * w, f[7] * w));
      }
    }
  } else {
    for (int c = tid; c < a.rows_ld; c += kRtThreads) {
      const float x = c < a.width ? rf(src[c]) : 0.f;
      for (int k = 0; k < a.top; ++k) out[s_row[k] * a.rows_ld + c] = T(x * weight[k]);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128) expert_combine_kernel(const T* __restrict__ y, const int* __restrict__ place,
                                                             T* __restrict__ out, int64_t y_ld, int64_t out_ld, int top,
                                                             int width) {
  const int64_t t = blockIdx.x;
  constexpr int V = sizeof(T) == 2 ? 8 : 4;  // width is a multiple of 8
  for (int c = threadIdx.x * V; c < width; c += 128 * V) {
    float s[V];
#pragma unroll
    for (int i = 0; i < V; ++i) s[i] = 0.f;
    for (int k = 0; k < top; ++k) {
      const int64_t row = place != nullptr ? place[t * top + k] : t * top + k;
      const uint4 u = *reinterpret_cast<const uint4*>(y + row * y_ld + c);
      const T* e = reinterpret_cast<const T*>(&u);
#pragma unroll
      for (int i = 0; i < V; ++i) s[i] += rf(e[i]);
    }
    uint4 o;
    T* e = reinterpret_cast<T*>(&o);
#pragma unroll
    for (int i = 0; i < V; ++i) e[i] = T(s[i]);
    *reinterpret_cast<uint4*>(out + t * out_ld + c) = o;
  }
}

namespace {

bool route_bad(const RouteArgs& a) {
  return a.tokens <= 0 || a.experts <= 0 || a.experts > kRtMaxExperts || a.top <= 0 || a.top > a.experts || a.width <= 0 ||
         a.rows_ld < a.width || a.h_ld < a.width || a.logits_ld < a.experts || a.block <= 0 ||
         static_cast<int64_t>(a.tokens) * a.top > 0x3fffffff;
}

template <int EPL>
int launch_small(const RouteArgs& a, cudaStream_t stream) {
  const int want = (a.tokens * a.top + 1) / 2, grid = want < 148 ? want : 148;
  if (a.act_bf16)
    route_small_kernel<__nv_bfloat16, EPL><<<grid, kRsThreads, 0, stream>>>(a);
  else
    route_small_kernel<float, EPL><<<grid, kRsThreads, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <int EPL>
int launch_sort(const RouteArgs& a, cudaStream_t stream) {
  if (cudaMemsetAsync(a.counts, 0, sizeof(int) * a.experts, stream) != cudaSuccess) return -4;
  route_topk_kernel<EPL><<<(a.tokens + kRtTokens - 1) / kRtTokens, kRtThreads, sizeof(int) * a.experts, stream>>>(a);
  route_layout_kernel<<<1, kRtThreads, 0, stream>>>(a);
  if (a.act_bf16)
    route_gather_kernel<__nv_bfloat16><<<a.tokens, kRtThreads, sizeof(int) * a.top, stream>>>(a);
  else
    route_gather_kernel<float><<<a.tokens, kRtThreads, sizeof(int) * a.top, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace
}  // namespace axb

// At most 1024 pairs and experts: offsets, row_pair and rows_out (block 1).
extern "C" int axb_route_small(const axb::RouteArgs* args, cudaStream_t stream) {
  const axb::RouteArgs& a = *args;
  if (axb::route_bad(a) || a.block != 1 || a.tokens * a.top > axb::kRtMaxPairs) return -10;
  if (a.experts <= 64) return axb::launch_small<2>(a, stream);
  if (a.experts <= 256) return axb::launch_small<8>(a, stream);
  return axb::launch_small<32>(a, stream);
}

// Any number of pairs: ids, weight, place, offsets, block_expert (block > 1) or row_pair (block 1), rows_out.
// Rows between the runs are not written.
extern "C" int axb_route_sort(const axb::RouteArgs* args, cudaStream_t stream) {
  const axb::RouteArgs& a = *args;
  if (axb::route_bad(a) || a.ids == nullptr || a.weight == nullptr || a.counts == nullptr) return -10;
  if (a.experts <= 64) return axb::launch_sort<2>(a, stream);
  if (a.experts <= 256) return axb::launch_sort<8>(a, stream);
  return axb::launch_sort<32>(a, stream);
}

// out[t, :width] = sum_k y[place[t * top + k], :width] (place null: rows in pair order); width, pitches multiples of 8.
extern "C" int axb_expert_combine(const void* y, const int* place, void* out, int64_t tokens, int64_t y_ld,
                                  int64_t out_ld, int top, int width, int act_bf16, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (width <= 0 || (width % 8) || (y_ld % 8) || (out_ld % 8) || top <= 0) return -10;
  if (act_bf16)
    axb::expert_combine_kernel<__nv_bfloat16><<<static_cast<unsigned>(tokens), 128, 0, stream>>>(
        static_cast<const __nv_bfloat16*>(y), place, static_cast<__nv_bfloat16*>(out), y_ld, out_ld, top, width);
  else
    axb::expert_combine_kernel<float><<<static_cast<unsigned>(tokens), 128, 0, stream>>>(
        static_cast<const float*>(y), place, static_cast<float*>(out), y_ld, out_ld, top, width);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
