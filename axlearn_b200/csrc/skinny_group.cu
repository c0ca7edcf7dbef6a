// A few rows times many small matrices, every group of rows with its own: out[r, n] = sum_k x[r, k] w[g][n, k].
//
// Groups are heads (every row meets every matrix: `offsets` null, x and out advance by x_group / out_group
// elements per group) or experts (group g owns rows [offsets[g], offsets[g + 1])).  Row r of the result goes
// to row row_out[r] (null: r).  With a gate the result is gate(x w[n], x w[up_off + n]).
//
//   skinny_mma_kernel   bf16 with 16-byte aligned rows.  The weights are the bound: every lane reads them as
//                       16-byte pieces straight into mma fragments (the contraction order is permuted the
//                       same way on both sides, so that a lane's eight consecutive values fill its slots of
//                       two k16 steps), 16 weight rows per CTA, its warps share the contraction.
//   skinny_plain_kernel any sizes and alignment, fp32 or bf16: a warp per weight row.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "gate_math.cuh"
#include "mma_sync.cuh"

namespace axb {

struct SkinnyArgs {
  const void* x;
  const void* w;
  void* out;
  const int* offsets;   // [groups + 1] or null
  const int* row_out;   // or null
  int64_t x_row, x_group, w_row, w_group, out_row, out_group;
  int rows, groups, n, k, up_off;
  int gate_kind;        // GateKind, -1: none
  int act_bf16;
  float limit, alpha;
};

namespace {

__device__ __forceinline__ float kf(float x) { return x; }
__device__ __forceinline__ float kf(__nv_bfloat16 x) { return __bfloat162float(x); }

__device__ __forceinline__ float apply_gate(const SkinnyArgs& a, float g, float u) {
  switch (a.gate_kind) {
    case kGateSilu: return gate_value<kGateSilu>(g, u, a.limit, a.alpha);
    case kGateGeluTanh: return gate_value<kGateGeluTanh>(g, u, a.limit, a.alpha);
    default: return gate_value<kGateClamped>(g, u, a.limit, a.alpha);
  }
}

__device__ __forceinline__ uint4 ldg_stream(const __nv_bfloat16* p) {
  uint4 r;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(r.x), "=r"(r.y), "=r"(r.z), "=r"(r.w) : "l"(p));
  return r;
}

constexpr int kSkWarps = 4, kSkThreads = 32 * kSkWarps;

}  // namespace

// RT tiles of 8 rows per pass; kGate: two weight rows per result.
template <int RT, bool kGate>
__global__ void __launch_bounds__(kSkThreads) skinny_mma_kernel(SkinnyArgs a) {
  using bf16 = __nv_bfloat16;
  constexpr int G = kGate ? 2 : 1;
  __shared__ float red[kSkWarps][G][16][RT * 8 + 1];
  const int n0 = blockIdx.x * 16, g = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lq = lane & 3;
  int lo = 0, hi = a.rows;
  if (a.offsets != nullptr) lo = a.offsets[g], hi = a.offsets[g + 1];
  lo += blockIdx.z * RT * 8;
  if (lo >= hi) return;
  const bf16* w = static_cast<const bf16*>(a.w) + g * a.w_group;
  const bf16* x = static_cast<const bf16*>(a.x) + g * a.x_group;
  bf16* out = static_cast<bf16*>(a.out) + g * a.out_group;
  // Weight rows of this lane; rows beyond n read row 0 and are not stored.
  const bf16* wp[G][2];
#pragma unroll
  for (int q = 0; q < G; ++q)
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int n = n0 + lr + u * 8;
      wp[q][u] = w + static_cast<int64_t>(n < a.n ? n + q * a.up_off : 0) * a.w_row + lq * 8;
    }
  for (int r0 = lo; r0 < hi; r0 += gridDim.z * RT * 8) {
    const bf16* xp[RT];
#pragma unroll
    for (int t = 0; t < RT; ++t) xp[t] = x + static_cast<int64_t>(min(r0 + t * 8 + lr, hi - 1)) * a.x_row + lq * 8;
    float acc[G][RT][4];
#pragma unroll
    for (int q = 0; q < G; ++q)
#pragma unroll
      for (int t = 0; t < RT; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[q][t][e] = 0.f;
    constexpr int kUnroll = RT >= 4 ? 2 : 4;
#pragma unroll 1
    for (int k0 = warp * 32; k0 < a.k; k0 += kSkWarps * 32 * kUnroll) {
      uint4 wf[kUnroll][G][2], xf[kUnroll][RT];
#pragma unroll
      for (int i = 0; i < kUnroll; ++i) {
        const int k = k0 + i * kSkWarps * 32;
        const bool in = k + lq * 8 < a.k;  // k is a multiple of 8
#pragma unroll
        for (int q = 0; q < G; ++q)
#pragma unroll
          for (int u = 0; u < 2; ++u) wf[i][q][u] = in ? ldg_stream(wp[q][u] + k) : make_uint4(0, 0, 0, 0);
#pragma unroll
        for (int t = 0; t < RT; ++t)
          xf[i][t] = in ? *reinterpret_cast<const uint4*>(xp[t] + k) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
      for (int i = 0; i < kUnroll; ++i)
#pragma unroll
        for (int q = 0; q < G; ++q) {
          const uint32_t a0[4] = {wf[i][q][0].x, wf[i][q][1].x, wf[i][q][0].y, wf[i][q][1].y};
          const uint32_t a1[4] = {wf[i][q][0].z, wf[i][q][1].z, wf[i][q][0].w, wf[i][q][1].w};
#pragma unroll
          for (int t = 0; t < RT; ++t) {
            mma(acc[q][t], a0, xf[i][t].x, xf[i][t].y);
            mma(acc[q][t], a1, xf[i][t].z, xf[i][t].w);
          }
        }
    }
    __syncthreads();  // the previous pass has been stored
#pragma unroll
    for (int q = 0; q < G; ++q)
#pragma unroll
      for (int t = 0; t < RT; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) red[warp][q][lr + (e >> 1) * 8][t * 8 + lq * 2 + (e & 1)] = acc[q][t][e];
    __syncthreads();
    for (int i = tid; i < 16 * RT * 8; i += kSkThreads) {
      const int n = i % 16, c = i / 16, r = r0 + c;
      if (n0 + n >= a.n || r >= hi) continue;
      float y[G];
#pragma unroll
      for (int q = 0; q < G; ++q) {
        y[q] = 0.f;
#pragma unroll
        for (int v = 0; v < kSkWarps; ++v) y[q] += red[v][q][n][c];
      }
      const int64_t dst = a.row_out != nullptr ? a.row_out[r] : r;
      out[dst * a.out_row + n0 + n] = __float2bfloat16(kGate ? apply_gate(a, y[0], y[G - 1]) : y[0]);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) skinny_plain_kernel(SkinnyArgs a) {
  const int n = blockIdx.x * 8 + (threadIdx.x >> 5), g = blockIdx.y, lane = threadIdx.x & 31;
  if (n >= a.n) return;
  int lo = 0, hi = a.rows;
  if (a.offsets != nullptr) lo = a.offsets[g], hi = a.offsets[g + 1];
  const T* w = static_cast<const T*>(a.w) + g * a.w_group + static_cast<int64_t>(n) * a.w_row;
  const T* up = w + static_cast<int64_t>(a.up_off) * a.w_row;
  const T* x = static_cast<const T*>(a.x) + g * a.x_group;
  T* out = static_cast<T*>(a.out) + g * a.out_group;
  for (int r = lo + blockIdx.z; r < hi; r += gridDim.z) {
    const T* row = x + static_cast<int64_t>(r) * a.x_row;
    float y = 0.f, u = 0.f;
    for (int k = lane; k < a.k; k += 32) {
      const float v = kf(row[k]);
      y += v * kf(w[k]);
      if (a.gate_kind >= 0) u += v * kf(up[k]);
    }
    for (int off = 16; off > 0; off >>= 1) {
      y += __shfl_xor_sync(0xffffffffu, y, off);
      u += __shfl_xor_sync(0xffffffffu, u, off);
    }
    if (lane == 0) {
      const int64_t dst = a.row_out != nullptr ? a.row_out[r] : r;
      out[dst * a.out_row + n] = T(a.gate_kind >= 0 ? apply_gate(a, y, u) : y);
    }
  }
}

template <int RT>
static int launch_skinny(const SkinnyArgs& a, int passes, cudaStream_t stream) {
  const dim3 grid((a.n + 15) / 16, a.groups, passes);
  if (a.gate_kind >= 0)
    skinny_mma_kernel<RT, true><<<grid, kSkThreads, 0, stream>>>(a);
  else
    skinny_mma_kernel<RT, false><<<grid, kSkThreads, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace axb

extern "C" int axb_skinny_group(const axb::SkinnyArgs* args, cudaStream_t stream) {
  using namespace axb;
  const SkinnyArgs& a = *args;
  if (a.rows <= 0 || a.n <= 0) return 0;
  if (a.groups <= 0 || a.groups > 65535 || a.k <= 0 || a.gate_kind > kGateClamped || a.up_off < 0) return -10;
  const uintptr_t bytes = reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.w);
  const bool aligned = !((a.x_row | a.x_group | a.w_row | a.w_group | a.k) & 7) && !(bytes & 15);
  if (a.act_bf16 && aligned) {
    // Rows a group has on average (experts) or exactly (heads).
    const int per = a.offsets != nullptr ? (a.rows + a.groups - 1) / a.groups : a.rows;
    if (per <= 8) return launch_skinny<1>(a, 1, stream);
    if (per <= 16) return launch_skinny<2>(a, 1, stream);
    const int passes = a.offsets != nullptr ? 1 : (a.rows + 31) / 32;
    return launch_skinny<4>(a, passes < 1024 ? passes : 1024, stream);
  }
  const int spread = a.offsets != nullptr ? 4 : (a.rows < 256 ? a.rows : 256);
  const dim3 grid((a.n + 7) / 8, a.groups, spread);
  if (a.act_bf16)
    skinny_plain_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(a);
  else
    skinny_plain_kernel<float><<<grid, 256, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
