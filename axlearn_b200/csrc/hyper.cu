// Hyper-connections: write of one sublayer, read and norm of the next, in one pass over the rows.
//
// One CTA per token row.  The S residual streams of the row (fp32) are read once, mixed with the
// branch, written once; the read-out u of the next sublayer stays in shared memory between the pass
// that computes it and the pass that writes norm(u).  A branch made of two RMS-normed outputs takes one
// more pass over those two (half-width) rows for their mean squares.
//
//   y     = branch                                         (one output)
//         = w * (rms(a) * sa + rms(b) * sb)                (two outputs, rms with its own eps)
//   x_t  <- sum_s mix[s, t] x_s + m * out[t] * y           (skipped without a branch; mix = null: identity,
//                                                           out = null: ones)
//   u     = sum_s read[s] x_s                              (read = null: plain sum)
//   h     = u / sqrt(mean(u^2) + eps) * (offset + scale) * h_mult   (scale = null: h = u, fp32)
//
// All arithmetic is fp32.  `h` rows are h_ld wide and zero beyond the width.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace axb {

struct HyperArgs {
  const void* streams;   // [rows, ld] one copy (streams_equal) or fp32 [rows, S, D]
  const void* branch_a;
  const void* branch_b;
  const float* scale_a;
  const float* scale_b;
  const float* mix;      // [S, S] from, to, or null
  const float* out_w;    // [S] or null
  const float* read;     // [S] or null
  const float* norm_scale;
  float* streams_out;    // [rows, S, D] or null
  void* h;
  int64_t rows, streams_ld, branch_ld, h_ld;
  int width, num_streams, streams_equal, streams_bf16, act_bf16;
  float multiplier, pair_weight, pair_eps, eps, norm_offset, h_mult;
};

constexpr int kMaxStreams = 16;

template <int V>
struct Vec {
  float v[V];
};

template <int V>
__device__ __forceinline__ Vec<V> load_vec(const float* p) {
  Vec<V> r;
  if (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    r.v[0] = f.x, r.v[1 % V] = f.y, r.v[2 % V] = f.z, r.v[3 % V] = f.w;
  } else {
    r.v[0] = p[0];
  }
  return r;
}
template <int V>
__device__ __forceinline__ Vec<V> load_vec(const __nv_bfloat16* p) {
  Vec<V> r;
  if (V == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162&>(u.x));
    const float2 b = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162&>(u.y));
    r.v[0] = a.x, r.v[1 % V] = a.y, r.v[2 % V] = b.x, r.v[3 % V] = b.y;
  } else {
    r.v[0] = __bfloat162float(p[0]);
  }
  return r;
}
template <int V>
__device__ __forceinline__ void store_vec(float* p, const Vec<V>& r) {
  if (V == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1 % V], r.v[2 % V], r.v[3 % V]);
  } else {
    p[0] = r.v[0];
  }
}
template <int V>
__device__ __forceinline__ void store_vec(__nv_bfloat16* p, const Vec<V>& r) {
  if (V == 4) {
    uint2 u;
    reinterpret_cast<__nv_bfloat162&>(u.x) = __floats2bfloat162_rn(r.v[0], r.v[1 % V]);
    reinterpret_cast<__nv_bfloat162&>(u.y) = __floats2bfloat162_rn(r.v[2 % V], r.v[3 % V]);
    *reinterpret_cast<uint2*>(p) = u;
  } else {
    p[0] = __float2bfloat16(r.v[0]);
  }
}

// Sums of two values over the CTA; every thread gets both.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* scratch) {
  for (int off = 16; off > 0; off >>= 1) {
    a += __shfl_xor_sync(0xffffffffu, a, off);
    b += __shfl_xor_sync(0xffffffffu, b, off);
  }
  const int warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) scratch[warp] = make_float2(a, b);
  __syncthreads();
  float2 s = make_float2(0.f, 0.f);
  for (int w = 0; w < warps; ++w) s.x += scratch[w].x, s.y += scratch[w].y;
  return s;
}

// TS: element type of the incoming streams; T: branches and output; S: compile-time stream count (0 =
// run-time, up to kMaxStreams); V: elements per access.
constexpr int max_threads(int S) { return S >= 1 && S <= 4 ? 512 : 256; }

template <typename TS, typename T, int S, int V>
__global__ void __launch_bounds__(max_threads(S)) hyper_step_kernel(HyperArgs a) {
  extern __shared__ float u_row[];  // [width]
  __shared__ float2 scratch[32];
  __shared__ float s_mix[kMaxStreams * kMaxStreams], s_out[kMaxStreams], s_read[kMaxStreams];
  constexpr int SM = S ? S : kMaxStreams;
  const int n = S ? S : a.num_streams;
  const int64_t row = blockIdx.x;
  const bool has_branch = a.branch_a != nullptr;
  if (has_branch)
    for (int i = threadIdx.x; i < n * n; i += blockDim.x)
      s_mix[i] = a.mix != nullptr ? a.mix[i] : (i / n == i % n ? 1.f : 0.f);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    s_read[i] = a.read != nullptr ? a.read[i] : 1.f;
    s_out[i] = has_branch ? (a.out_w != nullptr ? a.out_w[i] : 1.f) * a.multiplier : 0.f;
  }
  __syncthreads();

  const T* ba = static_cast<const T*>(a.branch_a) + row * a.branch_ld;
  const T* bb = static_cast<const T*>(a.branch_b) + row * a.branch_ld;
  float ra = 0.f, rb = 0.f;
  if (a.branch_b != nullptr) {
    float qa = 0.f, qb = 0.f;
    for (int c = threadIdx.x * V; c < a.width; c += blockDim.x * V) {
      const Vec<V> x = load_vec<V>(ba + c), y = load_vec<V>(bb + c);
#pragma unroll
      for (int i = 0; i < V; ++i) qa += x.v[i] * x.v[i], qb += y.v[i] * y.v[i];
    }
    const float2 q = block_sum2(qa, qb, scratch);
    ra = a.pair_weight * rsqrtf(q.x / a.width + a.pair_eps);
    rb = a.pair_weight * rsqrtf(q.y / a.width + a.pair_eps);
  }

  const TS* xs = static_cast<const TS*>(a.streams) + row * a.streams_ld;
  float* xo = a.streams_out == nullptr ? nullptr : a.streams_out + row * n * a.width;
  float sq = 0.f;
  for (int c = threadIdx.x * V; c < a.width; c += blockDim.x * V) {
    Vec<V> x[SM];
    if (a.streams_equal) {
      const Vec<V> one = load_vec<V>(xs + c);
#pragma unroll
      for (int s = 0; s < SM; ++s) x[s] = one;
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < n) x[s] = load_vec<V>(xs + static_cast<int64_t>(s) * a.width + c);
    }
    Vec<V> u;
#pragma unroll
    for (int i = 0; i < V; ++i) u.v[i] = 0.f;
    if (has_branch) {
      Vec<V> y = load_vec<V>(ba + c);
      if (a.branch_b != nullptr) {
        const Vec<V> z = load_vec<V>(bb + c), wa = load_vec<V>(a.scale_a + c), wb = load_vec<V>(a.scale_b + c);
#pragma unroll
        for (int i = 0; i < V; ++i) y.v[i] = y.v[i] * ra * wa.v[i] + z.v[i] * rb * wb.v[i];
      }
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t < n) {
          Vec<V> o;
          const float w = s_out[t], r = s_read[t];
#pragma unroll
          for (int i = 0; i < V; ++i) o.v[i] = w * y.v[i];
#pragma unroll
          for (int s = 0; s < SM; ++s) {
            if (s < n) {
              const float m = s_mix[s * n + t];
#pragma unroll
              for (int i = 0; i < V; ++i) o.v[i] += m * x[s].v[i];
            }
          }
          if (xo != nullptr) store_vec<V>(xo + static_cast<int64_t>(t) * a.width + c, o);
#pragma unroll
          for (int i = 0; i < V; ++i) u.v[i] += r * o.v[i];
        }
      }
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s) {
        if (s < n) {
          const float r = s_read[s];
#pragma unroll
          for (int i = 0; i < V; ++i) u.v[i] += r * x[s].v[i];
        }
      }
    }
    if (a.norm_scale == nullptr) {
      store_vec<V>(static_cast<float*>(a.h) + row * a.h_ld + c, u);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) sq += u.v[i] * u.v[i];
      store_vec<V>(u_row + c, u);  // read back by the same thread only
    }
  }
  if (a.norm_scale == nullptr) return;
  const float inv = a.h_mult * rsqrtf(block_sum2(sq, 0.f, scratch).x / a.width + a.eps);
  T* ho = static_cast<T*>(a.h) + row * a.h_ld;
  for (int c = threadIdx.x * V; c < a.width; c += blockDim.x * V) {
    Vec<V> u = load_vec<V>(u_row + c);
    const Vec<V> w = load_vec<V>(a.norm_scale + c);
#pragma unroll
    for (int i = 0; i < V; ++i) u.v[i] *= inv * (a.norm_offset + w.v[i]);
    store_vec<V>(ho + c, u);
  }
  for (int c = a.width + threadIdx.x; c < a.h_ld; c += blockDim.x) ho[c] = T(0.f);
}

template <typename TS, typename T, int S, int V>
static int launch_hyper(const HyperArgs& a, cudaStream_t stream) {
  const int smem = a.width * static_cast<int>(sizeof(float));
  auto kernel = hyper_step_kernel<TS, T, S, V>;
  static int configured = 48 * 1024;
  if (smem > configured) {
    if (smem > 220 * 1024 ||
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return -3;
    configured = smem;
  }
  // Few rows (decoding): the whole row in flight at once; many rows: several CTAs per SM.
  const int want = (a.width / V + 31) / 32 * 32;
  const int cap = a.rows <= 512 ? max_threads(S) : 256;
  const int threads = want < 64 ? 64 : (want > cap ? cap : want);
  kernel<<<static_cast<unsigned>(a.rows), threads, smem, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename TS, typename T>
static int dispatch_hyper(const HyperArgs& a, cudaStream_t stream) {
  const bool v4 = a.width % 4 == 0 && a.streams_ld % 4 == 0 && a.branch_ld % 4 == 0 && a.h_ld % 4 == 0;
  if (!v4) return launch_hyper<TS, T, 0, 1>(a, stream);
  switch (a.num_streams) {
    case 1: return launch_hyper<TS, T, 1, 4>(a, stream);
    case 2: return launch_hyper<TS, T, 2, 4>(a, stream);
    case 3: return launch_hyper<TS, T, 3, 4>(a, stream);
    case 4: return launch_hyper<TS, T, 4, 4>(a, stream);
    case 6: return launch_hyper<TS, T, 6, 4>(a, stream);
    case 8: return launch_hyper<TS, T, 8, 4>(a, stream);
    default: return launch_hyper<TS, T, 0, 1>(a, stream);
  }
}

}  // namespace axb

// Returns 0, -10 for unsupported sizes.
extern "C" int axb_hyper_step(const axb::HyperArgs* args, cudaStream_t stream) {
  const axb::HyperArgs& a = *args;
  if (a.rows == 0) return 0;
  if (a.width <= 0 || a.num_streams < 1 || a.num_streams > axb::kMaxStreams || a.rows > 0x7fffffff) return -10;
  if (!a.streams_equal && a.streams_bf16) return -10;
  if (a.act_bf16) {
    if (a.streams_bf16) return axb::dispatch_hyper<__nv_bfloat16, __nv_bfloat16>(a, stream);
    return axb::dispatch_hyper<float, __nv_bfloat16>(a, stream);
  }
  if (a.streams_bf16) return axb::dispatch_hyper<__nv_bfloat16, float>(a, stream);
  return axb::dispatch_hyper<float, float>(a, stream);
}
