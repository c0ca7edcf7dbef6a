// Gated feed-forward activation on a packed (gate | up) product (gate_math.cuh has the kinds).
//
// fp32 arithmetic, bf16 or fp32 elements; any row pitch and up-column offset.  Output rows are out_ld wide
// and zero beyond F.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "gate_math.cuh"

namespace axb {

template <typename T, int K>
__global__ void gated_act_kernel(const T* __restrict__ gu, T* __restrict__ out, int64_t n, int F, int up_off,
                                 int64_t ld, int64_t out_ld, float limit, float alpha) {
  const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int64_t row = i / out_ld;
  const int c = static_cast<int>(i % out_ld);
  const T* p = gu + row * ld;
  out[i] = c < F ? T(gate_value<K>(float(p[c]), float(p[up_off + c]), limit, alpha)) : T(0.f);
}

template <int K>
__global__ void gated_act_vec_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ out, int64_t n8,
                                     int up_off, int64_t ld, int64_t out_ld, float limit, float alpha) {
  const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n8) return;
  const int64_t per_row = out_ld / 8, row = i / per_row;
  const int c = static_cast<int>(i % per_row) * 8;
  const uint4 g = *reinterpret_cast<const uint4*>(gu + row * ld + c);
  const uint4 u = *reinterpret_cast<const uint4*>(gu + row * ld + up_off + c);
  uint4 r;
  const uint32_t gw[4] = {g.x, g.y, g.z, g.w}, uw[4] = {u.x, u.y, u.z, u.w};
  uint32_t* rw = reinterpret_cast<uint32_t*>(&r);
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const float2 a = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162&>(gw[k]));
    const float2 b = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162&>(uw[k]));
    const __nv_bfloat162 y = __floats2bfloat162_rn(gate_value<K>(a.x, b.x, limit, alpha), gate_value<K>(a.y, b.y, limit, alpha));
    rw[k] = reinterpret_cast<const uint32_t&>(y);
  }
  *reinterpret_cast<uint4*>(out + row * out_ld + c) = r;
}

template <int K>
static int launch_gated_act(const void* gu, void* out, int64_t rows, int F, int up_off, int64_t ld, int64_t out_ld,
                            int act_bf16, float limit, float alpha, cudaStream_t stream) {
  if (act_bf16 && F % 8 == 0 && up_off % 8 == 0 && ld % 8 == 0 && out_ld == F) {
    const int64_t n8 = rows * (F / 8);
    gated_act_vec_kernel<K><<<static_cast<unsigned>((n8 + 255) / 256), 256, 0, stream>>>(
        static_cast<const __nv_bfloat16*>(gu), static_cast<__nv_bfloat16*>(out), n8, up_off, ld, out_ld, limit, alpha);
  } else {
    const int64_t n = rows * out_ld;
    const unsigned grid = static_cast<unsigned>((n + 255) / 256);
    if (act_bf16)
      gated_act_kernel<__nv_bfloat16, K><<<grid, 256, 0, stream>>>(
          static_cast<const __nv_bfloat16*>(gu), static_cast<__nv_bfloat16*>(out), n, F, up_off, ld, out_ld, limit, alpha);
    else
      gated_act_kernel<float, K><<<grid, 256, 0, stream>>>(static_cast<const float*>(gu), static_cast<float*>(out), n, F,
                                                           up_off, ld, out_ld, limit, alpha);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace axb

// gu [rows, ld]: gate columns [0, F), up columns [up_off, up_off + F); out [rows, out_ld].  kind: GateKind;
// limit and alpha belong to the clamped kind.
extern "C" int axb_gated_act(const void* gu, void* out, int64_t rows, int F, int up_off, int64_t ld, int64_t out_ld,
                             int act_bf16, int kind, float limit, float alpha, cudaStream_t stream) {
  using namespace axb;
  if (rows <= 0) return 0;
  if (F <= 0 || up_off < F || ld < up_off + F || out_ld < F) return -10;
  switch (kind) {
    case kGateSilu:
      return launch_gated_act<kGateSilu>(gu, out, rows, F, up_off, ld, out_ld, act_bf16, limit, alpha, stream);
    case kGateGeluTanh:
      return launch_gated_act<kGateGeluTanh>(gu, out, rows, F, up_off, ld, out_ld, act_bf16, limit, alpha, stream);
    case kGateClamped:
      return launch_gated_act<kGateClamped>(gu, out, rows, F, up_off, ld, out_ld, act_bf16, limit, alpha, stream);
    default:
      return -10;
  }
}
