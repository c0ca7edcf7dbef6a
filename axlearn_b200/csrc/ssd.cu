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
//   ssd_norm_kernel      the group norm over the gated outputs `v`.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

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
  void* v;               // [B, T, inner] gated outputs ahead of the norm
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
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
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
      for (int i = 0; i < V; ++i) acc[i] = silu_f(acc[i]);
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
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
#pragma unroll
    for (int j = 0; j < K - 1; ++j)
#pragma unroll
      for (int i = 0; i < V; ++i) x[j][i] = x[j + 1][i];
    load_v<V>(src + t * a.ld, x[K - 1]);
    float acc[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      acc[i] = bias[i];
#pragma unroll
      for (int j = 0; j < K; ++j) acc[i] += w[j][i] * x[j][i];
      acc[i] = silu_f(acc[i]);
    }
    store_v<V>(dst + t * a.xbc_ld, acc);
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

// rms of v over one norm group, times the weight; columns [inner, out_ld) are written as zeros.
template <typename T, int V>
__global__ void __launch_bounds__(256) ssd_norm_kernel(SsdArgs a) {
  const int inner = a.heads * a.vdim, width = inner / a.norm_groups, c0 = blockIdx.y * width;
  const int64_t row = blockIdx.x;
  const T* v = static_cast<const T*>(a.v) + row * inner + c0;
  T* out = static_cast<T*>(a.out) + row * a.out_ld + c0;
  __shared__ float red[8];
  float sq = 0.f;
  for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
    float f[V];
    load_v<V>(v + c, f);
#pragma unroll
    for (int i = 0; i < V; ++i) sq += f[i] * f[i];
  }
  for (int off = 16; off > 0; off >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, off);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) total += red[w];
  const float inv = rsqrtf(total / width + a.eps);
  for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
    float f[V];
    load_v<V>(v + c, f);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] *= inv * a.norm_w[c0 + c + i];
    store_v<V>(out + c, f);
  }
  if (blockIdx.y == 0) {
    T* whole = static_cast<T*>(a.out) + row * a.out_ld;
    for (int c = inner + threadIdx.x; c < a.out_ld; c += blockDim.x) whole[c] = T(0.f);
  }
}

constexpr int kSdThreads = 256;

// V = 4: vdim is a multiple of 4; V = 1: any vdim.
template <typename T, int V>
__global__ void __launch_bounds__(kSdThreads) ssd_decode_kernel(SsdArgs a) {
  extern __shared__ float sm[];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int P = a.vdim, N = a.state, inner = a.heads * P, channels = ssd_channels(a);
  T* vout = static_cast<T*>(a.v) + static_cast<int64_t>(b) * inner + h * P;
  if (ssd_inactive(a, b)) {
    for (int c = tid; c < P; c += kSdThreads) vout[c] = T(0.f);
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
  const int pos = a.start[b], group = h / (a.heads / a.groups);
  const bool owns_bc = h % (a.heads / a.groups) == 0;
  T* ring = static_cast<T*>(a.ring) + static_cast<int64_t>(b) * a.taps * channels;
  const float dt = softplus_f(sf(row[a.dt_off + h]) + a.dt_bias[h]);
  const float decay = expf(-expf(a.a_log[h]) * dt);
  for (int i = tid; i < P + 2 * N; i += kSdThreads) {
    const int c = i < P ? h * P + i : (i < P + N ? inner + group * N + i - P : inner + a.groups * N + group * N + i - P - N);
    const T cur = row[a.xbc_off + c];
    float acc = a.conv_b[c] + a.conv_w[static_cast<int64_t>(a.taps - 1) * channels + c] * sf(cur);
    for (int j = 1; j < a.taps && j <= pos; ++j)
      acc += a.conv_w[static_cast<int64_t>(a.taps - 1 - j) * channels + c] *
             sf(ring[static_cast<int64_t>((pos - j) % a.taps) * channels + c]);
    if (i < P || owns_bc) ring[static_cast<int64_t>(pos % a.taps) * channels + c] = cur;
    acc = silu_f(acc);
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
    vout[p] = T(y * silu_f(sf(row[a.z_off + h * P + p])));
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
  T* vout = static_cast<T*>(a.v) + static_cast<int64_t>(b) * a.T * inner + h * P;
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
      const float z = sf(proj[(t0 + t) * a.ld + a.z_off + h * P + p0 + c]);
      vout[static_cast<int64_t>(t0 + t) * inner + p0 + c] = T(y * silu_f(z));
    }
  }
  for (int i = tid; i < (a.T - live) * kSsCols; i += kSsThreads) {
    const int c = i % kSsCols;
    if (p0 + c < P) vout[static_cast<int64_t>(live + i / kSsCols) * inner + p0 + c] = T(0.f);
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
// The products C_i . B_j belong to a GROUP, so a CTA takes four units of 16 value columns of one group's
// heads (one warp each, of the same or of different heads) and computes them once.  Every warp then forms
// its head's weights in registers.  For a tile of 16 x 16 pairs below the diagonal the decay splits at the
// end r of the token tile ahead of i's: exp(G_i - G_r) exp(G_r - G_j), both at most one, so no decay strength
// overflows and the exponentials are per token, not per pair; on the diagonal it is formed per pair.
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

constexpr int kScTok = 64, kScThreads = 128, kScWarps = 4;
constexpr float kL2e = 1.4426950408889634f;

template <int NP>
struct ScSmem {
  static constexpr int kNP = NP + 8, kXP = 24, kCP = 72;
  static constexpr int kB = 0;                                  // bf16 [64][kNP]
  static constexpr int kC = kB + kScTok * kNP * 2;              // bf16 [64][kNP]
  static constexpr int kX = kC + kScTok * kNP * 2;              // bf16 [4][64][kXP]
  static constexpr int kCB = kX + kScWarps * kScTok * kXP * 2;  // float [64][kCP]
  static constexpr int kG = kCB + kScTok * kCP * 4;             // float [4][64] running log2 decay
  static constexpr int kDt = kG + kScWarps * kScTok * 4;        // float [4][64]
  static constexpr int kF = kDt + kScWarps * kScTok * 4;        // float [4][4][64]: dt_j exp(G_(16 r + 15) - G_j)
  static constexpr int kTotal = kF + kScWarps * 4 * kScTok * 4;
};

}  // namespace

template <int NP, bool kStateOnly>
__global__ void __launch_bounds__(kScThreads, 3) ssd_chunk_kernel(SsdArgs a) {
  using L = ScSmem<NP>;
  using bf16 = __nv_bfloat16;
  constexpr int NT = NP / 8;
  extern __shared__ __align__(16) uint8_t ssd_smem[];
  bf16* sB = reinterpret_cast<bf16*>(ssd_smem + L::kB);
  bf16* sC = reinterpret_cast<bf16*>(ssd_smem + L::kC);
  float* sCB = reinterpret_cast<float*>(ssd_smem + L::kCB);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lc = (lane & 3) * 2;
  bf16* sX = reinterpret_cast<bf16*>(ssd_smem + L::kX) + warp * kScTok * L::kXP;
  float* sG = reinterpret_cast<float*>(ssd_smem + L::kG) + warp * kScTok;
  float* sDt = reinterpret_cast<float*>(ssd_smem + L::kDt) + warp * kScTok;
  float* sF = reinterpret_cast<float*>(ssd_smem + L::kF) + warp * 4 * kScTok;

  const int P = a.vdim, N = a.state, inner = a.heads * P, hpg = a.heads / a.groups, pt = (P + 15) / 16;
  const int tiles = (hpg * pt + kScWarps - 1) / kScWarps;
  const int seg = blockIdx.x, group = blockIdx.y / tiles, b = blockIdx.z;
  const int unit = (blockIdx.y % tiles) * kScWarps + warp;
  const bool owner = unit < hpg * pt;
  const int h = group * hpg + (owner ? unit / pt : 0), p0 = owner ? (unit % pt) * 16 : 0;
  const int pcols = owner ? min(16, P - p0) : 0;
  const bool inactive = ssd_inactive(a, b);
  const int live = inactive ? 0 : ssd_live(a, b);
  const int t_lo = seg * a.seg_tokens, t_hi = a.segments > 1 ? min(a.T, t_lo + a.seg_tokens) : a.T;
  const bf16* xbc = static_cast<const bf16*>(a.xbc) + static_cast<int64_t>(b) * a.T * a.xbc_ld;
  const bf16* proj = static_cast<const bf16*>(a.proj) + static_cast<int64_t>(b) * a.T * a.ld;
  bf16* vout = static_cast<bf16*>(a.v) + static_cast<int64_t>(b) * a.T * inner + h * P + p0;
  const int b_off = inner + group * N, c_off = b_off + a.groups * N;
  const bool vec_bc = !((a.xbc_ld | b_off | c_off | N) & 7), vec_x = !((a.xbc_ld | P) & 7);
  const bool pairs = !((P | a.z_off | a.ld | inner) & 1);
  const float rate = owner ? -expf(a.a_log[h]) * kL2e : 0.f, dt_bias = owner ? a.dt_bias[h] : 0.f;
  const float skip = owner ? a.d[h] : 0.f;

  // State, transposed: row = value column, column = state channel.
  float S[NT][4];
  const bool segmented = a.segments > 1;
  float* state = a.ssm + (static_cast<int64_t>(b) * a.heads + h) * N * P;
  float* seg_state =
      segmented ? a.seg_state + ((static_cast<int64_t>(b) * a.heads + h) * a.segments + seg) * N * P : nullptr;
  const float* init = segmented ? seg_state : state;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int p = lr + (e >> 1) * 8, c = n * 8 + lc + (e & 1);
      S[n][e] = !kStateOnly && p < pcols && c < N ? init[static_cast<int64_t>(c) * P + p0 + p] : 0.f;
    }
  float decay_sum = 0.f;

  for (int t0 = t_lo; t0 < t_hi; t0 += kScTok) {
    const int rows = max(0, min(kScTok, min(live, t_hi) - t0));
    if (rows == 0) {  // nothing live here or later in this segment: zero the outputs
      if (!kStateOnly) {
        const int n = min(kScTok, t_hi - t0);
        for (int i = lane; i < n * 16; i += 32)
          if (i % 16 < pcols) vout[static_cast<int64_t>(t0 + i / 16) * inner + i % 16] = __float2bfloat16(0.f);
      }
      continue;
    }
    __syncthreads();  // everybody is done with the previous chunk's tiles
    const bf16* src = xbc + static_cast<int64_t>(t0) * a.xbc_ld;
    auto load_bc = [&](bf16* tile, int off) {
      constexpr int kPer = NP / 8, kStep = kScThreads / kPer;
      const int c = (tid % kPer) * 8;
#pragma unroll
      for (int r = tid / kPer; r < kScTok; r += kStep) {
        bf16* dst = tile + r * L::kNP + c;
        const bf16* p = src + r * a.xbc_ld + off + c;
        if (vec_bc && r < rows && c < N) {
          cp16(dst, p);
        } else if (vec_bc || r >= rows || c >= N) {
          *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        } else {
#pragma unroll 1
          for (int e = 0; e < 8; ++e) dst[e] = c + e < N ? p[e] : __float2bfloat16(0.f);
        }
      }
    };
    load_bc(sB, b_off);
    if (!kStateOnly) load_bc(sC, c_off);
#pragma unroll
    for (int i = 0; i < 4; ++i) {  // the warp's own 64 x 16 slice of x
      const int r = i * 16 + (lane >> 1), c = (lane & 1) * 8;
      bf16* dst = sX + r * L::kXP + c;
      const bf16* p = src + r * a.xbc_ld + h * P + p0 + c;
      if (vec_x && r < rows && c < pcols) {
        cp16(dst, p);
      } else if (vec_x || r >= rows || c >= pcols) {
        *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
      } else {
#pragma unroll 1
        for (int e = 0; e < 8; ++e) dst[e] = c + e < pcols ? p[e] : __float2bfloat16(0.f);
      }
    }
    cp_commit();

    // Gates of this warp's outputs (rows lr + 8 k), as bf16 pairs.
    uint32_t z[8][2];
    if (!kStateOnly) {
#pragma unroll
      for (int m = 0; m < 8; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const int r = m * 8 + lr, c = n * 8 + lc;
          z[m][n] = 0;
          if (r < rows && c < pcols) {
            const bf16* p = proj + (t0 + r) * a.ld + a.z_off + h * P + p0 + c;
            if (pairs) {
              z[m][n] = *reinterpret_cast<const uint32_t*>(p);
            } else {
              __nv_bfloat162 q = __halves2bfloat162(p[0], c + 1 < pcols ? p[1] : p[0]);
              z[m][n] = reinterpret_cast<uint32_t&>(q);
            }
          }
        }
    }
    // Step sizes and running log decays of the warp's head: lane holds tokens lane and lane + 32.
    {
      float dt[2], g[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = lane + 32 * i;
        dt[i] = owner && r < rows ? softplus_f(__bfloat162float(proj[(t0 + r) * a.ld + a.dt_off + h]) + dt_bias) : 0.f;
        g[i] = rate * dt[i];
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
          const float y = __shfl_up_sync(0xffffffffu, g[i], off);
          if (lane >= off) g[i] += y;
        }
      }
      g[1] += __shfl_sync(0xffffffffu, g[0], 31);
      const float ref[4] = {__shfl_sync(0xffffffffu, g[0], 15), __shfl_sync(0xffffffffu, g[0], 31),
                            __shfl_sync(0xffffffffu, g[1], 15), __shfl_sync(0xffffffffu, g[1], 31)};
      decay_sum += ref[3];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = lane + 32 * i;
        sG[r] = g[i];
        sDt[r] = dt[i];
#pragma unroll
        for (int q = kStateOnly ? 3 : 0; q < 4; ++q) sF[q * kScTok + r] = r < 16 * (q + 1) ? dt[i] * ex2(ref[q] - g[i]) : 0.f;
      }
    }
    cp_wait_all();
    __syncthreads();

    float O[4][2][4];
    if (!kStateOnly) {
      // Products C_i . B_j of the ten 16 x 16 tiles on and below the diagonal, shared out over the warps.
      for (int tile = warp; tile < 10; tile += kScWarps) {
        const int m = tile < 1 ? 0 : tile < 3 ? 1 : tile < 6 ? 2 : 3, n = tile - m * (m + 1) / 2;
        float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int k = 0; k < NP; k += 16) {
          uint32_t af[4], bf[4];
          ldsm4(af, sC + (m * 16 + (lane & 15)) * L::kNP + k + (lane >> 4) * 8);
          ldsm4(bf, sB + (n * 16 + (lane >> 4) * 8 + (lane & 7)) * L::kNP + k + ((lane >> 3) & 1) * 8);
          mma(c0, af, bf[0], bf[1]);
          mma(c1, af, bf[2], bf[3]);
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          float* dst = sCB + (m * 16 + lr + half * 8) * L::kCP + n * 16 + lc;
          *reinterpret_cast<float2*>(dst) = make_float2(c0[half * 2], c0[half * 2 + 1]);
          *reinterpret_cast<float2*>(dst + 8) = make_float2(c1[half * 2], c1[half * 2 + 1]);
        }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) O[m][n][e] = 0.f;
      // O = C S_in: the state's accumulators as B fragments, hi and lo.
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
          for (int u = 0; u < 2; ++u) {
            mma(O[m][u], af, bh[u][0], bh[u][1]);
            mma(O[m][u], af, bl[u][0], bl[u][1]);
          }
        }
      }
      __syncthreads();  // all products are in shared memory
      uint32_t bx[4][4];
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) ldsm4t(bx[kk], sX + (kk * 16 + (lane & 15)) * L::kXP + (lane >> 4) * 8);
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const int r0 = m * 16 + lr, r1 = r0 + 8;
        const float g0 = sG[r0], g1 = sG[r1];
        const float e0 = ex2(g0), e1 = ex2(g1);
#pragma unroll
        for (int n = 0; n < 2; ++n) O[m][n][0] *= e0, O[m][n][1] *= e0, O[m][n][2] *= e1, O[m][n][3] *= e1;
        const float ref = m > 0 ? sG[m > 0 ? m * 16 - 1 : 0] : 0.f;
        const float d0 = ex2(g0 - ref), d1 = ex2(g1 - ref);
#pragma unroll
        for (int kk = 0; kk <= m; ++kk) {
          uint32_t ah[4], al[4];
#pragma unroll
          for (int q = 0; q < 2; ++q) {  // columns kk * 16 + q * 8 + lc, + 1
            const int c = kk * 16 + q * 8 + lc;
            const float2 s0 = *reinterpret_cast<const float2*>(sCB + r0 * L::kCP + c);
            const float2 s1 = *reinterpret_cast<const float2*>(sCB + r1 * L::kCP + c);
            float2 w0, w1;
            if (kk < m) {
              const float2 f = *reinterpret_cast<const float2*>(sF + (m > 0 ? m - 1 : 0) * kScTok + c);
              w0 = make_float2(d0 * f.x, d0 * f.y), w1 = make_float2(d1 * f.x, d1 * f.y);
            } else {
              const float2 g = *reinterpret_cast<const float2*>(sG + c), dt = *reinterpret_cast<const float2*>(sDt + c);
              w0 = make_float2(c <= r0 ? ex2(g0 - g.x) * dt.x : 0.f, c + 1 <= r0 ? ex2(g0 - g.y) * dt.y : 0.f);
              w1 = make_float2(c <= r1 ? ex2(g1 - g.x) * dt.x : 0.f, c + 1 <= r1 ? ex2(g1 - g.y) * dt.y : 0.f);
            }
            split2(s0.x * w0.x, s0.y * w0.y, ah[2 * q], al[2 * q]);
            split2(s1.x * w1.x, s1.y * w1.y, ah[2 * q + 1], al[2 * q + 1]);
          }
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            mma(O[m][n], ah, bx[kk][2 * n], bx[kk][2 * n + 1]);
            mma(O[m][n], al, bx[kk][2 * n], bx[kk][2 * n + 1]);
          }
        }
      }
    }
    // S = exp(G_63) S + (w x)^T B with w_j = dt_j exp(G_63 - G_j), hi and lo.
    {
      const float end = ex2(sG[kScTok - 1]);
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[n][e] *= end;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t ax[4], ah[4], al[4];
        ldsm4t(ax, sX + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * L::kXP + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const float2 w = *reinterpret_cast<const float2*>(sF + 3 * kScTok + kk * 16 + q * 8 + lc);
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const float2 x = unpack2(ax[2 * q + u]);
            split2(x.x * w.x, x.y * w.y, ah[2 * q + u], al[2 * q + u]);
          }
        }
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
          uint32_t bf[4];
          ldsm4t(bf, sB + (kk * 16 + (lane & 15)) * L::kNP + n * 8 + (lane >> 4) * 8);
          mma(S[n], ah, bf[0], bf[1]);
          mma(S[n + 1], ah, bf[2], bf[3]);
          mma(S[n], al, bf[0], bf[1]);
          mma(S[n + 1], al, bf[2], bf[3]);
        }
      }
    }
    if (kStateOnly) continue;
    const int n_out = min(kScTok, t_hi - t0);
#pragma unroll
    for (int m = 0; m < 8; ++m)
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int r = m * 8 + lr, c = n * 8 + lc;
        if (r < n_out && c < pcols) {
          const float2 x = unpack2(*reinterpret_cast<const uint32_t*>(sX + r * L::kXP + c)), g = unpack2(z[m][n]);
          float y0 = 0.f, y1 = 0.f;
          if (r < rows) {
            y0 = (O[m >> 1][n][(m & 1) * 2] + skip * x.x) * __fdividef(g.x, 1.f + ex2(-g.x * kL2e));
            y1 = (O[m >> 1][n][(m & 1) * 2 + 1] + skip * x.y) * __fdividef(g.y, 1.f + ex2(-g.y * kL2e));
          }
          bf16* dst = vout + static_cast<int64_t>(t0 + r) * inner + c;
          if (pairs) {
            *reinterpret_cast<uint32_t*>(dst) = pack2(y0, y1);
          } else {
            dst[0] = __float2bfloat16(y0);
            if (c + 1 < pcols) dst[1] = __float2bfloat16(y1);
          }
        }
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
      if (p < pcols && c < N) dst[static_cast<int64_t>(c) * P + p0 + p] = S[n][e];
    }
  if (kStateOnly && owner && p0 == 0 && lane == 0)
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
  for (int g = 0; g < a.segments; ++g) {
    float* p = a.seg_state + (bh * a.segments + g) * n + i;
    const float add = *p;
    *p = s;
    s = s * exp2f(a.seg_decay[bh * a.segments + g]) + add;
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
  const int units = a.heads / a.groups * ((a.vdim + 15) / 16);
  const int tiles = (units + kScWarps - 1) / kScWarps;
  kernel<<<dim3(a.segments, a.groups * tiles, a.B), kScThreads, smem, stream>>>(a);
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
  const bool vec = !((width | inner | static_cast<int>(a.out_ld)) & 7);
  const int want = ((vec ? width / 8 : width) + 31) / 32 * 32;
  const int threads = want < 32 ? 32 : (want > 256 ? 256 : want);
  const dim3 grid(static_cast<unsigned>(rows), a.norm_groups);
  if (vec)
    ssd_norm_kernel<T, 8><<<grid, threads, 0, stream>>>(a);
  else
    ssd_norm_kernel<T, 1><<<grid, threads, 0, stream>>>(a);
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

// Gated outputs into a.v, token by token; needs a.xbc.  state <= 512.
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
