// State-space duality (Mamba-2): matrix state per head, one scalar decay per token.
//
// Columns of a token's projection row ([B, T, ld]): z [inner] | x, B, C [inner + 2 G N] | dt [H], inner = H P.
//   x, B, C  <- silu(causal conv, `taps` taps per channel, + bias)
//   dt       <- softplus(dt + dt_bias)
//   S_t = exp(-exp(a_log) dt_t) S_(t-1) + dt_t B_t x_t^T       [N, P], fp32 (head h: group h / (H / G))
//   y_t = S_t^T C_t + d x_t
//   out = rms over norm_groups equal parts of (y silu(z)) * norm_w
//
// `start[b]` tokens have been seen (null: zero; < 0: row not in this step), `live[b]` of the T new ones are
// valid (null: T).  The state [B, H, N, P] and the ring of convolution inputs [B, taps, channels] (position p
// in slot p % taps) are updated in place.
//
//   ssd_conv_kernel      prompts: convolution and silu of all channels; ssd_ring_kernel then stores the last
//                        inputs (a launch of its own: the convolution still reads the old ones).
//   ssd_chunk_kernel     bf16 prompts: chunks of 64 tokens on the tensor cores (see there).
//   ssd_scan_kernel      token by token with the state in registers: fp32, and large states.
//   ssd_decode_kernel    one token per sequence: convolution, state update and read-out; streams the state
//                        once.  The ring slot that is written is not one that the step reads.
//   ssd_norm_kernel      gate and group norm of the outputs `y`.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include <type_traits>

#include "mma_sync.cuh"

namespace axb {

struct SsdArgs {
  const void* proj;
  const float* conv_w;   // [taps, channels]
  const float* conv_b;
  const float* dt_bias;  // [H]
  const float* a_log;    // [H]
  const float* d;        // [H]
  const float* norm_w;   // [inner]
  float* ssm;            // [B, H, N, P]
  void* ring;            // [B, taps, channels]
  void* xbc;             // [B, T, xbc_ld] convolved channels (prompts)
  void* y;               // [B, T, inner] outputs ahead of the gate
  void* out;             // [B, T, out_ld]
  float* seg_state;      // [B, H, segments, N, P] (segmented prompts)
  float* seg_decay;      // [B, H, segments], log2
  const int* start;
  const int* live;
  int64_t ld, xbc_ld, out_ld;
  int B, T, heads, vdim, state, groups, taps, norm_groups;
  int z_off, xbc_off, dt_off, act_bf16, segments, seg_tokens;
  float eps;
};

namespace {

__device__ __forceinline__ float sf(float x) { return x; }
__device__ __forceinline__ float sf(__nv_bfloat16 x) { return __bfloat162float(x); }
// x * sigmoid(x); of bf16 activations to well below their rounding.
__device__ __forceinline__ float silu_t(float x, float) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_t(float x, __nv_bfloat16) {
  return __fdividef(x, 1.f + ex2(-x * 1.4426950408889634f));
}
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ bool ssd_inactive(const SsdArgs& a, int b) {
  return (a.start != nullptr && a.start[b] < 0) || (a.live != nullptr && a.live[b] <= 0);
}
__device__ __forceinline__ int ssd_live(const SsdArgs& a, int b) {
  return a.live != nullptr ? min(a.live[b], a.T) : a.T;
}
__device__ __forceinline__ int ssd_channels(const SsdArgs& a) { return a.heads * a.vdim + 2 * a.groups * a.state; }

template <int V>
__device__ __forceinline__ void load_v(const __nv_bfloat16* p, float (&f)[V]) {
  if (V == 8) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 t = unpack2(w[i]);
      f[(2 * i) % V] = t.x, f[(2 * i + 1) % V] = t.y;
    }
  } else {
    f[0] = __bfloat162float(p[0]);
  }
}
template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&f)[V]) {
#pragma unroll
  for (int i = 0; i < V; i += 4) {
    if (V % 4 == 0) {
      const float4 u = *reinterpret_cast<const float4*>(p + i);
      f[i] = u.x, f[(i + 1) % V] = u.y, f[(i + 2) % V] = u.z, f[(i + 3) % V] = u.w;
    } else {
      f[0] = p[0];
    }
  }
}
template <int V>
__device__ __forceinline__ void store_v(__nv_bfloat16* p, const float (&f)[V]) {
  if (V == 8) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack2(f[0], f[1 % V]), pack2(f[2 % V], f[3 % V]), pack2(f[4 % V], f[5 % V]),
                                              pack2(f[6 % V], f[7 % V]));
  } else {
    p[0] = __float2bfloat16(f[0]);
  }
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float (&f)[V]) {
#pragma unroll
  for (int i = 0; i < V; ++i) p[i] = f[i];
}

constexpr int kConvThreads = 128, kConvTokens = 16;

}  // namespace

// TAPS > 0: that many taps in registers, V channels per thread, a run of 16 tokens.  TAPS = 0: any number.
template <typename T, int TAPS, int V>
__global__ void __launch_bounds__(kConvThreads) ssd_conv_kernel(SsdArgs a) {
  const int channels = ssd_channels(a);
  const int c = (blockIdx.x * kConvThreads + threadIdx.x) * V, b = blockIdx.z, t0 = blockIdx.y * kConvTokens;
  if (c >= channels || ssd_inactive(a, b)) return;
  const int taps = TAPS ? TAPS : a.taps;
  const int start = a.start != nullptr ? a.start[b] : 0;
  const T* src = static_cast<const T*>(a.proj) + static_cast<int64_t>(b) * a.T * a.ld + a.xbc_off + c;
  const T* ring = static_cast<const T*>(a.ring) + static_cast<int64_t>(b) * taps * channels + c;
  T* dst = static_cast<T*>(a.xbc) + static_cast<int64_t>(b) * a.T * a.xbc_ld + c;
  auto input = [&](int t, float (&f)[V]) {  // the input of token t, also of tokens before this block
    if (t >= 0) {
      load_v<V>(src + t * a.ld, f);
    } else if (start + t >= 0) {
      load_v<V>(ring + static_cast<int64_t>((start + t) % taps) * channels, f);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] = 0.f;
    }
  };
  float bias[V];
#pragma unroll
  for (int i = 0; i < V; ++i) bias[i] = a.conv_b[c + i];
  const int t1 = min(a.T, t0 + kConvTokens);
  if (TAPS == 0) {
    for (int t = t0; t < t1; ++t) {
      float acc[V], x[V];
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = bias[i];
      for (int j = 0; j < taps; ++j) {
        input(t - taps + 1 + j, x);
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] += a.conv_w[static_cast<int64_t>(j) * channels + c + i] * x[i];
      }
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = silu_t(acc[i], T(0.f));
      store_v<V>(dst + t * a.xbc_ld, acc);
    }
    return;
  }
  constexpr int K = TAPS ? TAPS : 1;
  float w[K][V], x[K][V];
#pragma unroll
  for (int j = 0; j < K; ++j)
#pragma unroll
    for (int i = 0; i < V; ++i) w[j][i] = a.conv_w[static_cast<int64_t>(j) * channels + c + i];
#pragma unroll
  for (int j = 0; j < K - 1; ++j) input(t0 - K + 1 + j, x[j + 1]);
  auto one = [&](int t) {  // x[K - 1] holds the token's input
    float acc[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      acc[i] = bias[i];
#pragma unroll
      for (int j = 0; j < K; ++j) acc[i] += w[j][i] * x[j][i];
      acc[i] = silu_t(acc[i], T(0.f));
    }
    store_v<V>(dst + t * a.xbc_ld, acc);
  };
  auto shift = [&]() {
#pragma unroll
    for (int j = 0; j < K - 1; ++j)
#pragma unroll
      for (int i = 0; i < V; ++i) x[j][i] = x[j + 1][i];
  };
  constexpr int kBatch = 8;  // tokens whose loads are in flight together
  int t = t0;
  if (sizeof(T) == 2 && V == 8) {
    for (; t + kBatch <= t1; t += kBatch) {
      uint4 raw[kBatch];
#pragma unroll
      for (int u = 0; u < kBatch; ++u) raw[u] = *reinterpret_cast<const uint4*>(src + (t + u) * a.ld);
#pragma unroll
      for (int u = 0; u < kBatch; ++u) {
        shift();
        const uint32_t r[4] = {raw[u].x, raw[u].y, raw[u].z, raw[u].w};
#pragma unroll
        for (int i = 0; i < V / 2; ++i) {
          const float2 f = unpack2(r[i % 4]);
          x[K - 1][2 * i] = f.x, x[K - 1][2 * i + 1] = f.y;
        }
        one(t + u);
      }
    }
  }
  for (; t < t1; ++t) {
    shift();
    load_v<V>(src + t * a.ld, x[K - 1]);
    one(t);
  }
}

template <typename T>
__global__ void ssd_ring_kernel(SsdArgs a) {
  const int channels = ssd_channels(a);
  const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
  if (c >= channels || ssd_inactive(a, b)) return;
  const int start = a.start != nullptr ? a.start[b] : 0, live = ssd_live(a, b);
  const T* src = static_cast<const T*>(a.proj) + static_cast<int64_t>(b) * a.T * a.ld + a.xbc_off + c;
  T* ring = static_cast<T*>(a.ring) + static_cast<int64_t>(b) * a.taps * channels + c;
  for (int t = max(0, live - a.taps); t < live; ++t) ring[static_cast<int64_t>((start + t) % a.taps) * channels] = src[t * a.ld];
}

// y silu(z), its rms over one norm group, times the weight; columns [inner, out_ld) are written as zeros.  NV > 0:
// a thread holds its NV vectors between the two passes; NV = 0: any width, computed twice.
template <typename T, int V, int NV>
__global__ void __launch_bounds__(256) ssd_norm_kernel(SsdArgs a) {
  const int inner = a.heads * a.vdim, width = inner / a.norm_groups, c0 = blockIdx.y * width;
  const int64_t row = blockIdx.x;
  const T* y = static_cast<const T*>(a.y) + row * inner + c0;
  const T* z = static_cast<const T*>(a.proj) + row * a.ld + a.z_off + c0;
  T* out = static_cast<T*>(a.out) + row * a.out_ld + c0;
  __shared__ float red[8];
  auto gated = [&](int c, float (&f)[V]) {
    float g[V];
    load_v<V>(y + c, f);
    load_v<V>(z + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] *= silu_t(g[i], T(0.f));
  };
  auto write = [&](int c, float (&f)[V], float inv) {
    float w[V];
    load_v<V>(a.norm_w + c0 + c, w);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] *= inv * w[i];
    store_v<V>(out + c, f);
  };
  float sq = 0.f;
  float keep[NV ? NV : 1][V];
  if (NV) {
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = (k * blockDim.x + threadIdx.x) * V;
      if (c < width) {
        gated(c, keep[k]);
#pragma unroll
        for (int i = 0; i < V; ++i) sq += keep[k][i] * keep[k][i];
      }
    }
  } else {
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
      gated(c, keep[0]);
#pragma unroll
      for (int i = 0; i < V; ++i) sq += keep[0][i] * keep[0][i];
    }
  }
  for (int off = 16; off > 0; off >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, off);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) total += red[w];
  const float inv = rsqrtf(total / width + a.eps);
  if (NV) {
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = (k * blockDim.x + threadIdx.x) * V;
      if (c < width) write(c, keep[k], inv);
    }
  } else {
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
      gated(c, keep[0]);
      write(c, keep[0], inv);
    }
  }
  if (blockIdx.y == 0) {
    T* whole = static_cast<T*>(a.out) + row * a.out_ld;
    for (int c = inner + threadIdx.x; c < a.out_ld; c += blockDim.x) whole[c] = T(0.f);
  }
}

constexpr int kSdThreads = 256;

// V = 4: vdim is a multiple of 4; V = 1: any vdim.
template <typename T, int V>
__global__ void __launch_bounds__(kSdThreads, 4) ssd_decode_kernel(SsdArgs a) {
  extern __shared__ float sm[];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int P = a.vdim, N = a.state, inner = a.heads * P, channels = ssd_channels(a);
  T* yout = static_cast<T*>(a.y) + static_cast<int64_t>(b) * inner + h * P;
  if (ssd_inactive(a, b)) {
    for (int c = tid; c < P; c += kSdThreads) yout[c] = T(0.f);
    return;
  }
  const int nc = (P + V - 1) / V;
  const int cols = min(nc, kSdThreads), groups = kSdThreads / cols, rg = tid / cols;
  float* S = a.ssm + (static_cast<int64_t>(b) * a.heads + h) * N * P;
  // The first rows of the state are on their way while the convolution is computed.
  constexpr int kAhead = 8;
  float s[kAhead][V];
  const int cv0 = tid % cols;
  if (rg < groups) {
#pragma unroll
    for (int u = 0; u < kAhead; ++u)
      if (rg + u * groups < N) {
        float* e = S + static_cast<int64_t>(rg + u * groups) * P + cv0 * V;
        load_v<V>(e, s[u]);
      }
  }
  float* s_x = sm;        // [P]
  float* s_b = s_x + P;   // [N], times dt
  float* s_c = s_b + N;   // [N]
  float* s_o = s_c + N;   // [row groups][P]
  const T* row = static_cast<const T*>(a.proj) + static_cast<int64_t>(b) * a.ld;
  const int pos = a.start[b], here = pos % a.taps, group = h / (a.heads / a.groups);
  const bool owns_bc = h % (a.heads / a.groups) == 0;
  T* ring = static_cast<T*>(a.ring) + static_cast<int64_t>(b) * a.taps * channels;
  const float dt = softplus_f(sf(row[a.dt_off + h]) + a.dt_bias[h]);
  const float decay = expf(-expf(a.a_log[h]) * dt);
  for (int i = tid; i < P + 2 * N; i += kSdThreads) {
    const int c = i < P ? h * P + i : (i < P + N ? inner + group * N + i - P : inner + a.groups * N + group * N + i - P - N);
    const T cur = row[a.xbc_off + c];
    float acc = a.conv_b[c] + a.conv_w[static_cast<int64_t>(a.taps - 1) * channels + c] * sf(cur);
    for (int j = 1, slot = here; j < a.taps && j <= pos; ++j) {
      slot = slot == 0 ? a.taps - 1 : slot - 1;
      acc += a.conv_w[static_cast<int64_t>(a.taps - 1 - j) * channels + c] * sf(ring[static_cast<int64_t>(slot) * channels + c]);
    }
    if (i < P || owns_bc) ring[static_cast<int64_t>(here) * channels + c] = cur;
    acc = silu_t(acc, T(0.f));
    sm[i] = i >= P && i < P + N ? acc * dt : acc;
  }
  __syncthreads();
  if (rg < groups) {
    for (int cv = cv0; cv < nc; cv += cols) {
      float x[V], o[V];
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] = s_x[cv * V + i], o[i] = 0.f;
      for (int n0 = rg; n0 < N; n0 += kAhead * groups) {
        if (cv != cv0 || n0 != rg) {
#pragma unroll
          for (int u = 0; u < kAhead; ++u)
            if (n0 + u * groups < N) {
              float* e = S + static_cast<int64_t>(n0 + u * groups) * P + cv * V;
              load_v<V>(e, s[u]);
            }
        }
#pragma unroll
        for (int u = 0; u < kAhead; ++u) {
          const int n = n0 + u * groups;
          if (n < N) {
            const float bn = s_b[n], cn = s_c[n];
            float* e = S + static_cast<int64_t>(n) * P + cv * V;
#pragma unroll
            for (int i = 0; i < V; ++i) {
              s[u][i] = decay * s[u][i] + bn * x[i];
              o[i] += cn * s[u][i];
            }
            if (V == 4) {
              *reinterpret_cast<float4*>(e) = make_float4(s[u][0], s[u][1 % V], s[u][2 % V], s[u][3 % V]);
            } else {
              e[0] = s[u][0];
            }
          }
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) s_o[rg * P + cv * V + i] = o[i];
    }
  }
  __syncthreads();
  for (int p = tid; p < P; p += kSdThreads) {
    float y = a.d[h] * s_x[p];
    for (int g = 0; g < groups; ++g) y += s_o[g * P + p];
    yout[p] = T(y);
  }
}

constexpr int kSsTok = 16, kSsCols = 32, kSsThreads = 256;

// State slice [N, 32] of one head in registers: thread (row group, column), RPT rows per thread.
template <typename T, int RPT>
__global__ void __launch_bounds__(kSsThreads) ssd_scan_kernel(SsdArgs a) {
  extern __shared__ float sm[];
  const int h = blockIdx.y, b = blockIdx.z, p0 = blockIdx.x * kSsCols;
  const int tid = threadIdx.x, rg = tid / kSsCols, col = tid % kSsCols;
  constexpr int RG = kSsThreads / kSsCols;
  const int P = a.vdim, N = a.state, inner = a.heads * P, group = h / (a.heads / a.groups);
  const int live = ssd_inactive(a, b) ? 0 : ssd_live(a, b);
  float* s_b = sm;                       // [16][N], times dt
  float* s_c = s_b + kSsTok * N;         // [16][N]
  float* s_x = s_c + kSsTok * N;         // [16][32]
  float* s_o = s_x + kSsTok * kSsCols;   // [16][RG][32]
  float* s_dt = s_o + kSsTok * kSsThreads;  // [16]
  float* s_al = s_dt + kSsTok;           // [16]
  const bool in = p0 + col < P;
  float* S = a.ssm + (static_cast<int64_t>(b) * a.heads + h) * N * P + p0 + col;
  float st[RPT];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int n = rg + r * RG;
    st[r] = live > 0 && in && n < N ? S[static_cast<int64_t>(n) * P] : 0.f;
  }
  const T* xbc = static_cast<const T*>(a.xbc) + static_cast<int64_t>(b) * a.T * a.xbc_ld;
  const T* proj = static_cast<const T*>(a.proj) + static_cast<int64_t>(b) * a.T * a.ld;
  T* yout = static_cast<T*>(a.y) + static_cast<int64_t>(b) * a.T * inner + h * P;
  const float rate = -expf(a.a_log[h]), skip = a.d[h];
  for (int t0 = 0; t0 < live; t0 += kSsTok) {
    const int n_tok = min(kSsTok, live - t0);
    __syncthreads();
    if (tid < n_tok) {
      const float dt = softplus_f(sf(proj[(t0 + tid) * a.ld + a.dt_off + h]) + a.dt_bias[h]);
      s_dt[tid] = dt;
      s_al[tid] = expf(rate * dt);
    }
    __syncthreads();
    for (int i = tid; i < n_tok * N; i += kSsThreads) {
      const int t = i / N, n = i % N;
      const T* row = xbc + (t0 + t) * a.xbc_ld + inner + group * N + n;
      s_b[i] = sf(row[0]) * s_dt[t];
      s_c[i] = sf(row[a.groups * N]);
    }
    for (int i = tid; i < n_tok * kSsCols; i += kSsThreads) {
      const int p = p0 + i % kSsCols;
      s_x[i] = p < P ? sf(xbc[(t0 + i / kSsCols) * a.xbc_ld + h * P + p]) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < n_tok; ++t) {
      const float x = s_x[t * kSsCols + col], al = s_al[t];
      float o = 0.f;
#pragma unroll
      for (int r = 0; r < RPT; ++r) {
        const int n = rg + r * RG;
        if (n < N) {
          st[r] = al * st[r] + s_b[t * N + n] * x;
          o += s_c[t * N + n] * st[r];
        }
      }
      s_o[(t * RG + rg) * kSsCols + col] = o;
    }
    __syncthreads();
    for (int i = tid; i < n_tok * kSsCols; i += kSsThreads) {
      const int t = i / kSsCols, c = i % kSsCols;
      if (p0 + c >= P) continue;
      float y = skip * s_x[i];
#pragma unroll
      for (int g = 0; g < RG; ++g) y += s_o[(t * RG + g) * kSsCols + c];
      yout[static_cast<int64_t>(t0 + t) * inner + p0 + c] = T(y);
    }
  }
  for (int i = tid; i < (a.T - live) * kSsCols; i += kSsThreads) {
    const int c = i % kSsCols;
    if (p0 + c < P) yout[static_cast<int64_t>(live + i / kSsCols) * inner + p0 + c] = T(0.f);
  }
  if (live <= 0) return;
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int n = rg + r * RG;
    if (in && n < N) S[static_cast<int64_t>(n) * P] = st[r];
  }
}

// ------------------------------------------------------------------------------------------
// Chunked form on the tensor cores.
// ------------------------------------------------------------------------------------------
//
// Within a chunk of 64 tokens let G_i be the running sum of the log decays (inclusive; base 2 here).
//   y_i   = exp(G_i) S_in^T C_i + sum_{j <= i} (C_i . B_j) exp(G_i - G_j) dt_j x_j
//   S_out = exp(G_63) S_in + sum_j exp(G_63 - G_j) dt_j B_j x_j^T
//
// One CTA = 4 warps per (64 value columns of a head, sequence, segment of the prompt).  The pair weights of a
// 16 x 16 tile come out of one warp's accumulators; below the diagonal their decay splits at the end r of the
// token tile ahead of i's: exp(G_i - G_r) exp(G_r - G_j), both at most one, so no decay strength overflows and
// the exponentials are per token, not per pair; on the diagonal they are formed per pair (which also takes the
// skip d x_i).  Everything else is split by value columns, 16 per warp.
//
// What enters the recurrence is kept to fp32 accuracy: pair weights, weighted x and the state as matrix
// operands are split into two bf16 terms; B, C and x are the bf16 outputs of the convolution.
//
// A warp holds its [16 value columns, N] of the state transposed as mma accumulators; in that layout the
// registers are the B fragments of the read-out S_in^T C.
//
// Long prompts of few sequences are cut into segments: a first launch (kStateOnly) computes what each
// segment alone adds to the state, ssd_segment_kernel chains them, and the second launch runs every segment
// from its true initial state.
namespace {

constexpr int kScTok = 64, kScCols = 64, kScThreads = 128;
constexpr float kL2e = 1.4426950408889634f;

template <int NP>
struct ScSmem {
  static constexpr int kNP = NP + 8, kXP = kScCols + 8;
  static constexpr int kB = 0;                             // bf16 [64][kNP]
  static constexpr int kC = kB + kScTok * kNP * 2;         // bf16 [64][kNP]
  static constexpr int kX = kC + kScTok * kNP * 2;         // bf16 [64][kXP]  x, then y
  static constexpr int kM = kX + kScTok * kXP * 2;         // bf16 [10 tiles][hi, lo][16][16]  pair weights
  static constexpr int kG = kM + 10 * 2 * 512;             // float [64] running log2 decay
  static constexpr int kDt = kG + kScTok * 4;              // float [64]
  static constexpr int kW = kDt + kScTok * 4;              // float [64]  dt_j exp(G_63 - G_j)
  static constexpr int kTotal = kW + kScTok * 4;
};

// S = exp(G_63) S + (w x)^T B with w_j = dt_j exp(G_63 - G_j), hi and lo; ax: x as A fragments (rows = value
// columns).
template <int NT>
__device__ __forceinline__ void update_state(float (&S)[NT][4], const uint32_t (&ax)[4][4], const __nv_bfloat16* sB,
                                             int pitch, const float* sG, const float* sW, int lane) {
  const int lc = (lane & 3) * 2;
  const float end = ex2(sG[kScTok - 1]);
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) S[n][e] *= end;
#pragma unroll
  for (int kk = 0; kk < 4; ++kk) {
    uint32_t ah[4], al[4];
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const float2 w = *reinterpret_cast<const float2*>(sW + kk * 16 + q * 8 + lc);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const float2 x = unpack2(ax[kk][2 * q + u]);
        split2(x.x * w.x, x.y * w.y, ah[2 * q + u], al[2 * q + u]);
      }
    }
#pragma unroll
    for (int n = 0; n < NT; n += 4) {
      uint32_t b0[4], b1[4];
      const __nv_bfloat16* p = sB + (kk * 16 + (lane & 15)) * pitch + n * 8 + (lane >> 4) * 8;
      ldsm4t(b0, p);
      ldsm4t(b1, p + 16);
      mma(S[n], ah, b0[0], b0[1]);
      mma(S[n + 1], ah, b0[2], b0[3]);
      mma(S[n + 2], ah, b1[0], b1[1]);
      mma(S[n + 3], ah, b1[2], b1[3]);
      mma(S[n], al, b0[0], b0[1]);
      mma(S[n + 1], al, b0[2], b0[3]);
      mma(S[n + 2], al, b1[0], b1[1]);
      mma(S[n + 3], al, b1[2], b1[3]);
    }
  }
}

}  // namespace

template <int NP, bool kStateOnly>
__global__ void __launch_bounds__(kScThreads, 4) ssd_chunk_kernel(SsdArgs a) {
  using L = ScSmem<NP>;
  using bf16 = __nv_bfloat16;
  constexpr int NT = NP / 8;
  extern __shared__ __align__(16) uint8_t ssd_smem[];
  bf16* sB = reinterpret_cast<bf16*>(ssd_smem + L::kB);
  bf16* sC = reinterpret_cast<bf16*>(ssd_smem + L::kC);
  bf16* sX = reinterpret_cast<bf16*>(ssd_smem + L::kX);
  uint8_t* sM = ssd_smem + L::kM;  // the 16-byte halves of a tile's rows swap places every four rows
  float* sG = reinterpret_cast<float*>(ssd_smem + L::kG);
  float* sDt = reinterpret_cast<float*>(ssd_smem + L::kDt);
  float* sW = reinterpret_cast<float*>(ssd_smem + L::kW);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lc = (lane & 3) * 2;

  const int P = a.vdim, N = a.state, inner = a.heads * P, blocks = (P + kScCols - 1) / kScCols;
  const int seg = blockIdx.x, h = blockIdx.y / blocks, p0 = (blockIdx.y % blocks) * kScCols, b = blockIdx.z;
  const int cols = min(kScCols, P - p0);                  // value columns of this CTA
  const int v0 = warp * 16, pcols = min(16, cols - v0);   // and of this warp (may be none)
  const int group = h / (a.heads / a.groups);
  const bool inactive = ssd_inactive(a, b);
  const int live = inactive ? 0 : ssd_live(a, b);
  const int t_lo = seg * a.seg_tokens, t_hi = a.segments > 1 ? min(a.T, t_lo + a.seg_tokens) : a.T;
  const int t_live = min(live, t_hi);
  const bf16* xbc = static_cast<const bf16*>(a.xbc) + static_cast<int64_t>(b) * a.T * a.xbc_ld;
  const bf16* dt_col = static_cast<const bf16*>(a.proj) + static_cast<int64_t>(b) * a.T * a.ld + a.dt_off + h;
  bf16* yout = static_cast<bf16*>(a.y) + static_cast<int64_t>(b) * a.T * inner + h * P + p0;
  const int x_off = h * P + p0, b_off = inner + group * N, c_off = b_off + a.groups * N;
  const bool vec_bc = !((a.xbc_ld | b_off | c_off | N) & 7), vec_x = !((a.xbc_ld | P | inner) & 7);
  const float rate = -expf(a.a_log[h]) * kL2e, dt_bias = a.dt_bias[h], skip = a.d[h];

  // State, transposed: row = value column, column = state channel.
  float S[NT][4];
  const bool segmented = a.segments > 1;
  float* state = a.ssm + (static_cast<int64_t>(b) * a.heads + h) * N * P + p0 + v0;
  float* seg_state =
      segmented ? a.seg_state + ((static_cast<int64_t>(b) * a.heads + h) * a.segments + seg) * N * P + p0 + v0 : nullptr;
  const float* init = segmented ? seg_state : state;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int p = lr + (e >> 1) * 8, c = n * 8 + lc + (e & 1);
      S[n][e] = !kStateOnly && p < pcols && c < N ? init[static_cast<int64_t>(c) * P + p] : 0.f;
    }
  float decay_sum = 0.f;
  // Step sizes of the coming chunk (warp 0: tokens lane and lane + 32).
  float raw[2] = {0.f, 0.f};
  auto fetch_dt = [&](int t0) {
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (t0 + lane + 32 * i < t_live) raw[i] = __bfloat162float(dt_col[static_cast<int64_t>(t0 + lane + 32 * i) * a.ld]);
  };
  if (warp == 0) fetch_dt(t_lo);

  for (int t0 = t_lo; t0 < t_hi; t0 += kScTok) {
    const int rows = max(0, min(kScTok, t_live - t0)), n_out = min(kScTok, t_hi - t0);
    if (rows == 0) {  // nothing live here or later in this segment: zero the outputs
      if (!kStateOnly)
        for (int i = tid; i < n_out * kScCols; i += kScThreads)
          if (i % kScCols < cols) yout[static_cast<int64_t>(t0 + i / kScCols) * inner + i % kScCols] = __float2bfloat16(0.f);
      continue;
    }
    __syncthreads();  // everybody is done with the previous chunk's tiles
    const bf16* src = xbc + static_cast<int64_t>(t0) * a.xbc_ld;
    // `width` columns of the chunk's rows into a tile of W columns, zero beyond.
    auto load_tile = [&](auto w_const, bf16* tile, int pitch, int off, int width, bool vec) {
      constexpr int W = decltype(w_const)::value, kPer = W / 8, kStep = kScThreads / kPer;
      const int c = (tid % kPer) * 8, r0 = tid / kPer;
      bf16* dst = tile + r0 * pitch + c;
      const bf16* p = src + r0 * a.xbc_ld + off + c;
      if (vec && c < width && rows == kScTok) {
#pragma unroll
        for (int i = 0; i < kScTok / kStep; ++i) {
          cp16(dst + i * kStep * pitch, p);
          p += kStep * a.xbc_ld;
        }
        return;
      }
#pragma unroll 1
      for (int r = r0; r < kScTok; r += kStep) {
        if (r >= rows || c >= width) {
          *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        } else if (vec) {
          cp16(dst, p);
        } else {
#pragma unroll 1
          for (int e = 0; e < 8; ++e) dst[e] = c + e < width ? p[e] : __float2bfloat16(0.f);
        }
        dst += kStep * pitch;
        p += kStep * a.xbc_ld;
      }
    };
    load_tile(std::integral_constant<int, NP>(), sB, L::kNP, b_off, N, vec_bc);
    if (!kStateOnly) load_tile(std::integral_constant<int, NP>(), sC, L::kNP, c_off, N, vec_bc);
    load_tile(std::integral_constant<int, kScCols>(), sX, L::kXP, x_off, cols, vec_x);
    cp_commit();
    // The next chunk's x starts its way from DRAM to L2 (B and C are shared by the heads of a group).
    if (tid >= 64 && t0 + tid < t_live) asm volatile("prefetch.global.L2 [%0];" ::"l"(src + tid * a.xbc_ld + x_off));

    if (warp == 0) {
      // Step sizes and running log decays.
      float dt[2], g[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        dt[i] = lane + 32 * i < rows ? softplus_f(raw[i] + dt_bias) : 0.f;
        g[i] = rate * dt[i];
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
          const float y = __shfl_up_sync(0xffffffffu, g[i], off);
          if (lane >= off) g[i] += y;
        }
      }
      g[1] += __shfl_sync(0xffffffffu, g[0], 31);
      const float end = __shfl_sync(0xffffffffu, g[1], 31);
      decay_sum += end;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        sG[lane + 32 * i] = g[i];
        sDt[lane + 32 * i] = dt[i];
        sW[lane + 32 * i] = dt[i] * ex2(end - g[i]);
      }
      fetch_dt(t0 + kScTok);
    }
    cp_wait_all();
    __syncthreads();

    if (!kStateOnly) {
      // Weights of the ten 16 x 16 tiles of pairs on and below the diagonal: a diagonal tile per warp, then the
      // other six.
#pragma unroll 1
      for (int tile = warp; tile < 10; tile += 4) {
        const int q = tile - 4;  // (1,0) (2,0) (2,1) (3,0) (3,1) (3,2)
        const int m = tile < 4 ? tile : q < 1 ? 1 : q < 3 ? 2 : 3, n = tile < 4 ? tile : q - m * (m - 1) / 2;
        float s[2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[u][e] = 0.f;
#pragma unroll
        for (int k = 0; k < NP; k += 16) {
          uint32_t af[4], bf[4];
          ldsm4(af, sC + (m * 16 + (lane & 15)) * L::kNP + k + (lane >> 4) * 8);
          ldsm4(bf, sB + (n * 16 + (lane >> 4) * 8 + (lane & 7)) * L::kNP + k + ((lane >> 3) & 1) * 8);
          mma(s[0], af, bf[0], bf[1]);
          mma(s[1], af, bf[2], bf[3]);
        }
        const int r0 = m * 16 + lr, r1 = r0 + 8;
        const float g0 = sG[r0], g1 = sG[r1];
        const float ref = sG[max(m * 16 - 1, 0)];
        const float d0 = ex2(g0 - ref), d1 = ex2(g1 - ref);  // off the diagonal
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int c = n * 16 + u * 8 + lc;
          const float2 g = *reinterpret_cast<const float2*>(sG + c), dt = *reinterpret_cast<const float2*>(sDt + c);
          float w[4];
          if (tile >= 4) {
            const float fx = dt.x * ex2(ref - g.x), fy = dt.y * ex2(ref - g.y);
            w[0] = s[u][0] * d0 * fx, w[1] = s[u][1] * d0 * fy, w[2] = s[u][2] * d1 * fx, w[3] = s[u][3] * d1 * fy;
          } else {
            w[0] = c <= r0 ? s[u][0] * ex2(g0 - g.x) * dt.x : 0.f;
            w[1] = c + 1 <= r0 ? s[u][1] * ex2(g0 - g.y) * dt.y : 0.f;
            w[2] = c <= r1 ? s[u][2] * ex2(g1 - g.x) * dt.x : 0.f;
            w[3] = c + 1 <= r1 ? s[u][3] * ex2(g1 - g.y) * dt.y : 0.f;
            if (c == r0) w[0] += skip;
            if (c + 1 == r0) w[1] += skip;
            if (c == r1) w[2] += skip;
            if (c + 1 == r1) w[3] += skip;
          }
          uint32_t hi, lo;
          uint8_t* at = sM + (m * (m + 1) / 2 + n) * 1024 + lr * 32 + (u ^ (lr >> 2 & 1)) * 16 + lc * 2;
          split2(w[0], w[1], hi, lo);
          *reinterpret_cast<uint32_t*>(at) = hi;
          *reinterpret_cast<uint32_t*>(at + 512) = lo;
          split2(w[2], w[3], hi, lo);
          *reinterpret_cast<uint32_t*>(at + 256) = hi;
          *reinterpret_cast<uint32_t*>(at + 768) = lo;
        }
      }
      // O = C S_in: the state's accumulators as B fragments, hi and lo.
      float O[4][2][4];
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) O[m][n][e] = 0.f;
#pragma unroll
      for (int kk = 0; kk < NP / 16; ++kk) {
        uint32_t bh[2][2], bl[2][2];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int t = 0; t < 2; ++t) split2(S[2 * kk + t][2 * u], S[2 * kk + t][2 * u + 1], bh[u][t], bl[u][t]);
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          uint32_t af[4];
          ldsm4(af, sC + (m * 16 + (lane & 15)) * L::kNP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
          for (int u = 0; u < 2; ++u) mma(O[m][u], af, bh[u][0], bh[u][1]);
#pragma unroll
          for (int u = 0; u < 2; ++u) mma(O[m][u], af, bl[u][0], bl[u][1]);
        }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const float e0 = ex2(sG[m * 16 + lr]), e1 = ex2(sG[m * 16 + lr + 8]);
#pragma unroll
        for (int n = 0; n < 2; ++n) O[m][n][0] *= e0, O[m][n][1] *= e0, O[m][n][2] *= e1, O[m][n][3] *= e1;
      }
      __syncthreads();  // all weights are in shared memory
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t bx[4];
        ldsm4t(bx, sX + (kk * 16 + (lane & 15)) * L::kXP + v0 + (lane >> 4) * 8);
#pragma unroll
        for (int m = kk; m < 4; ++m) {
          uint32_t ah[4], al[4];
          const uint8_t* at = sM + (m * (m + 1) / 2 + kk) * 1024 + (lane & 15) * 32 + ((lane >> 4) ^ (lane >> 2 & 1)) * 16;
          ldsm4(ah, at);
          ldsm4(al, at + 512);
          mma(O[m][0], ah, bx[0], bx[1]);
          mma(O[m][1], ah, bx[2], bx[3]);
          mma(O[m][0], al, bx[0], bx[1]);
          mma(O[m][1], al, bx[2], bx[3]);
        }
      }
      // The state's update reads x once more; y then takes its place (the warp's own columns).
      uint32_t ax[4][4];
#pragma unroll
      for (int kk = 0; kk < 4; ++kk)
        ldsm4t(ax[kk], sX + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * L::kXP + v0 + ((lane >> 3) & 1) * 8);
      __syncwarp();
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const int r = m * 16 + lr + half * 8;
            *reinterpret_cast<uint32_t*>(sX + r * L::kXP + v0 + n * 8 + lc) =
                r < rows ? pack2(O[m][n][half * 2], O[m][n][half * 2 + 1]) : 0u;
          }
      __syncwarp();
      update_state<NT>(S, ax, sB, L::kNP, sG, sW, lane);
      if (vec_x) {
        const int c = (lane & 1) * 8;
        if (c < pcols) {
          bf16* dst = yout + static_cast<int64_t>(t0 + (lane >> 1)) * inner + v0 + c;
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int r = i * 16 + (lane >> 1);
            if (r < n_out) *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(sX + r * L::kXP + v0 + c);
            dst += static_cast<int64_t>(16) * inner;
          }
        }
      } else {
        for (int i = lane; i < n_out * 16; i += 32)
          if (i % 16 < pcols) yout[static_cast<int64_t>(t0 + i / 16) * inner + v0 + i % 16] = sX[i / 16 * L::kXP + v0 + i % 16];
      }
    } else {
      uint32_t ax[4][4];
#pragma unroll
      for (int kk = 0; kk < 4; ++kk)
        ldsm4t(ax[kk], sX + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * L::kXP + v0 + ((lane >> 3) & 1) * 8);
      update_state<NT>(S, ax, sB, L::kNP, sG, sW, lane);
    }
  }

  // Final state: of the sequence (last segment), or of this segment alone.
  if (!kStateOnly && segmented && seg != a.segments - 1) return;
  if (inactive && !kStateOnly) return;
  float* dst = kStateOnly ? seg_state : state;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int p = lr + (e >> 1) * 8, c = n * 8 + lc + (e & 1);
      if (p < pcols && c < N) dst[static_cast<int64_t>(c) * P + p] = S[n][e];
    }
  if (kStateOnly && p0 == 0 && tid == 0)
    a.seg_decay[(static_cast<int64_t>(b) * a.heads + h) * a.segments + seg] = decay_sum;
}

// Chains the segments: on entry seg_state[s] is what segment s adds to a zero state, on exit the state
// at the segment's start.
__global__ void ssd_segment_kernel(SsdArgs a) {
  const int64_t bh = blockIdx.y;
  const int64_t n = static_cast<int64_t>(a.state) * a.vdim;
  const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  float s = a.ssm[bh * n + i];
  float* p = a.seg_state + bh * a.segments * n + i;
  constexpr int kBatch = 8;
  for (int g0 = 0; g0 < a.segments; g0 += kBatch) {
    float add[kBatch], decay[kBatch];
#pragma unroll
    for (int u = 0; u < kBatch; ++u)
      if (g0 + u < a.segments) {
        add[u] = p[(g0 + u) * n];
        decay[u] = a.seg_decay[bh * a.segments + g0 + u];
      }
#pragma unroll
    for (int u = 0; u < kBatch; ++u)
      if (g0 + u < a.segments) {
        p[(g0 + u) * n] = s;
        s = s * exp2f(decay[u]) + add[u];
      }
  }
}

namespace {

int launched() { return cudaGetLastError() == cudaSuccess ? 0 : -4; }

bool ssd_bad(const SsdArgs& a) {
  return a.B <= 0 || a.T <= 0 || a.heads <= 0 || a.vdim <= 0 || a.state <= 0 || a.groups <= 0 || a.heads % a.groups ||
         a.taps <= 0 || a.norm_groups <= 0 || (a.heads * a.vdim) % a.norm_groups || a.B > 65535 || a.heads > 65535 ||
         a.out_ld < static_cast<int64_t>(a.heads) * a.vdim;
}

template <typename T, int TAPS, int V>
int launch_conv(const SsdArgs& a, cudaStream_t stream) {
  const int channels = a.heads * a.vdim + 2 * a.groups * a.state;
  const dim3 grid((channels / V + kConvThreads - 1) / kConvThreads, (a.T + kConvTokens - 1) / kConvTokens, a.B);
  if (grid.y > 65535) return -10;
  ssd_conv_kernel<T, TAPS, V><<<grid, kConvThreads, 0, stream>>>(a);
  if (launched()) return -4;
  ssd_ring_kernel<T><<<dim3((channels + 255) / 256, a.B), 256, 0, stream>>>(a);
  return launched();
}

template <typename T>
int conv(const SsdArgs& a, cudaStream_t stream) {
  const int channels = a.heads * a.vdim + 2 * a.groups * a.state;
  if ((channels | a.xbc_off | a.ld | a.xbc_ld) & 7) return launch_conv<T, 0, 1>(a, stream);
  switch (a.taps) {
    case 2: return launch_conv<T, 2, 8>(a, stream);
    case 3: return launch_conv<T, 3, 8>(a, stream);
    case 4: return launch_conv<T, 4, 8>(a, stream);
    default: return launch_conv<T, 0, 8>(a, stream);
  }
}

template <typename T, int RPT>
int launch_scan(const SsdArgs& a, cudaStream_t stream) {
  const size_t smem = sizeof(float) * (2 * kSsTok * a.state + kSsTok * kSsCols + kSsTok * kSsThreads + 2 * kSsTok);
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    if (smem > 220 * 1024 || cudaFuncSetAttribute(ssd_scan_kernel<T, RPT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                  static_cast<int>(smem)) != cudaSuccess)
      return -3;
    configured = smem;
  }
  const dim3 grid((a.vdim + kSsCols - 1) / kSsCols, a.heads, a.B);
  ssd_scan_kernel<T, RPT><<<grid, kSsThreads, smem, stream>>>(a);
  return launched();
}

template <typename T>
int scan(const SsdArgs& a, cudaStream_t stream) {
  if (a.state <= 64) return launch_scan<T, 8>(a, stream);
  if (a.state <= 128) return launch_scan<T, 16>(a, stream);
  if (a.state <= 256) return launch_scan<T, 32>(a, stream);
  return launch_scan<T, 64>(a, stream);
}

template <typename T, int V>
int launch_decode(const SsdArgs& a, cudaStream_t stream) {
  const int nc = (a.vdim + V - 1) / V;
  const int groups = kSdThreads / (nc < kSdThreads ? nc : kSdThreads);
  const size_t smem = sizeof(float) * (a.vdim + 2 * a.state + static_cast<size_t>(groups) * a.vdim);
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    if (smem > 220 * 1024 || cudaFuncSetAttribute(ssd_decode_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                  static_cast<int>(smem)) != cudaSuccess)
      return -3;
    configured = smem;
  }
  ssd_decode_kernel<T, V><<<dim3(a.heads, a.B), kSdThreads, smem, stream>>>(a);
  return launched();
}

template <int NP, bool kStateOnly>
int launch_chunk_pass(const SsdArgs& a, cudaStream_t stream) {
  constexpr int smem = ScSmem<NP>::kTotal;
  auto kernel = ssd_chunk_kernel<NP, kStateOnly>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
    configured = true;
  }
  kernel<<<dim3(a.segments, a.heads * ((a.vdim + kScCols - 1) / kScCols), a.B), kScThreads, smem, stream>>>(a);
  return launched();
}

template <int NP>
int launch_chunk(const SsdArgs& a, cudaStream_t stream) {
  if (a.segments > 1) {
    const int rc = launch_chunk_pass<NP, true>(a, stream);
    if (rc) return rc;
    const int64_t n = static_cast<int64_t>(a.state) * a.vdim;
    ssd_segment_kernel<<<dim3(static_cast<unsigned>((n + 255) / 256), a.B * a.heads), 256, 0, stream>>>(a);
    if (launched()) return -4;
  }
  return launch_chunk_pass<NP, false>(a, stream);
}

template <typename T>
int norm(const SsdArgs& a, cudaStream_t stream) {
  const int inner = a.heads * a.vdim, width = inner / a.norm_groups;
  const int64_t rows = static_cast<int64_t>(a.B) * a.T;
  const bool vec = !((width | inner | a.z_off | static_cast<int>(a.out_ld | a.ld)) & 7);
  const int want = ((vec ? width / 8 : width) + 31) / 32 * 32;
  const int threads = want < 32 ? 32 : (want > 256 ? 256 : want);
  const dim3 grid(static_cast<unsigned>(rows), a.norm_groups);
  if (!vec)
    ssd_norm_kernel<T, 1, 0><<<grid, threads, 0, stream>>>(a);
  else if (width <= 8 * 256)
    ssd_norm_kernel<T, 8, 1><<<grid, threads, 0, stream>>>(a);
  else if (width <= 16 * 256)
    ssd_norm_kernel<T, 8, 2><<<grid, threads, 0, stream>>>(a);
  else if (width <= 32 * 256)
    ssd_norm_kernel<T, 8, 4><<<grid, threads, 0, stream>>>(a);
  else
    ssd_norm_kernel<T, 8, 0><<<grid, threads, 0, stream>>>(a);
  return launched();
}

}  // namespace
}  // namespace axb

// Prompts: convolved channels into a.xbc, last inputs into the ring.
extern "C" int axb_ssd_conv(const axb::SsdArgs* args, cudaStream_t stream) {
  const axb::SsdArgs& a = *args;
  if (axb::ssd_bad(a) || a.xbc == nullptr) return -10;
  return a.act_bf16 ? axb::conv<__nv_bfloat16>(a, stream) : axb::conv<float>(a, stream);
}

// Outputs into a.y, token by token; needs a.xbc.  state <= 512.
extern "C" int axb_ssd_scan(const axb::SsdArgs* args, cudaStream_t stream) {
  const axb::SsdArgs& a = *args;
  if (axb::ssd_bad(a) || a.xbc == nullptr || a.state > 512) return -10;
  return a.act_bf16 ? axb::scan<__nv_bfloat16>(a, stream) : axb::scan<float>(a, stream);
}

// The same in chunks: bf16, state <= 128.  segments > 1 needs seg_state / seg_decay and seg_tokens a multiple
// of 64 with segments * seg_tokens >= T.
extern "C" int axb_ssd_chunk(const axb::SsdArgs* args, cudaStream_t stream) {
  const axb::SsdArgs& a = *args;
  if (axb::ssd_bad(a) || !a.act_bf16 || a.xbc == nullptr || a.state > 128 || a.segments < 1) return -10;
  if (a.segments > 1 && (a.seg_state == nullptr || a.seg_decay == nullptr || a.seg_tokens % 64 ||
                         static_cast<int64_t>(a.segments) * a.seg_tokens < a.T))
    return -11;
  return a.state <= 64 ? axb::launch_chunk<64>(a, stream) : axb::launch_chunk<128>(a, stream);
}

// One token per sequence; needs a.start.
extern "C" int axb_ssd_decode(const axb::SsdArgs* args, cudaStream_t stream) {
  const axb::SsdArgs& a = *args;
  if (axb::ssd_bad(a) || a.T != 1 || a.start == nullptr) return -10;
  if (a.act_bf16)
    return a.vdim % 4 == 0 ? axb::launch_decode<__nv_bfloat16, 4>(a, stream) : axb::launch_decode<__nv_bfloat16, 1>(a, stream);
  return a.vdim % 4 == 0 ? axb::launch_decode<float, 4>(a, stream) : axb::launch_decode<float, 1>(a, stream);
}

extern "C" int axb_ssd_norm(const axb::SsdArgs* args, cudaStream_t stream) {
  const axb::SsdArgs& a = *args;
  if (axb::ssd_bad(a)) return -10;
  return a.act_bf16 ? axb::norm<__nv_bfloat16>(a, stream) : axb::norm<float>(a, stream);
}
