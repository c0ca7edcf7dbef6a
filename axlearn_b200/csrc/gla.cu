// Gated linear attention: a matrix-valued recurrent state, every key channel with its own decay.
//
// Per head, with q scaled by q_scale, key channel c and value column d:
//   z_t   = W_a2 (a1 of the projection) + bias              (low-rank gate, [heads * dim])
//   ld_t  = log sigmoid(z_t) / tau                          (log decay)
//   S_t   = diag(exp(ld_t)) S_(t-1) + k_t v_t^T             [dim, vdim], fp32
//   o_t   = S_t^T q_t
//   out   = o / sqrt(mean(o^2) + eps) * norm_w * silu(gate) (mean over vdim)
//
// q, k, v, gate and a1 are read from one packed projection row per token ([B, T, ld], element offsets).
// `start[b]` < 0 or `live[b]` <= 0: the row is not in this step.  Tokens at or beyond live[b] leave the
// state alone.  The state [B, heads, dim, vdim] is updated in place.
//
//   gla_decode_kernel  one token per sequence: streams the state once (read, decay, add, write) while
//                      accumulating o, then norm and gate; one CTA per (sequence, head).
//   gla_chunk_kernel   bf16 prompts: chunks of 64 tokens on the tensor cores (see there).
//   gla_scan_kernel    token by token with the state in registers: fp32, and sizes the chunk kernel
//                      does not take; followed by gla_norm_gate_kernel.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "mma_sync.cuh"

namespace axb {

struct GlaArgs {
  const void* proj;
  const void* a2;        // [heads * dim, rank]
  const float* a2_bias;  // [heads * dim]
  const float* norm_w;   // [vdim]
  float* state;          // [B, heads, dim, vdim]
  void* out;             // [B, T, out_ld]
  float* o_raw;          // [B, T, heads, vdim] un-normalised outputs (multi-slice, scan)
  float* seg_state;      // [B, heads, segments, dim, vdim] (segmented runs)
  float* seg_decay;      // [B, heads, segments, dim], log2
  const int* start;
  const int* live;
  int64_t ld, out_ld;
  int B, T, heads, dim, vdim, rank;
  int q_off, k_off, v_off, g_off, a1_off;
  int act_bf16, segments, seg_tokens;
  float inv_tau, q_scale, eps;
};

namespace {

__device__ __forceinline__ float gf(float x) { return x; }
__device__ __forceinline__ float gf(__nv_bfloat16 x) { return __bfloat162float(x); }

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }

__device__ __forceinline__ bool row_inactive(const GlaArgs& a, int b) {
  return (a.start != nullptr && a.start[b] < 0) || (a.live != nullptr && a.live[b] <= 0);
}
__device__ __forceinline__ int live_tokens(const GlaArgs& a, int b) {
  return a.live != nullptr ? min(a.live[b], a.T) : a.T;
}

constexpr int kGdThreads = 256;

}  // namespace

// V = 4: vdim is a multiple of 4 (vector accesses to the state); V = 1: any vdim.
template <typename T, int V>
__global__ void __launch_bounds__(kGdThreads) gla_decode_kernel(GlaArgs a) {
  extern __shared__ float sm[];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  T* out = static_cast<T*>(a.out) + static_cast<int64_t>(b) * a.out_ld + h * a.vdim;
  if (row_inactive(a, b)) {
    for (int c = tid; c < a.vdim; c += kGdThreads) out[c] = T(0.f);
    return;
  }
  float* s_q = sm;                 // [dim]
  float* s_k = s_q + a.dim;        // [dim]
  float* s_al = s_k + a.dim;       // [dim]
  float* s_a1 = s_al + a.dim;      // [rank]
  float* s_o = s_a1 + (a.rank + 3) / 4 * 4;  // [row groups][vdim]
  __shared__ float s_red[kGdThreads / 32];
  const T* row = static_cast<const T*>(a.proj) + static_cast<int64_t>(b) * a.ld;
  for (int r = tid; r < a.rank; r += kGdThreads) s_a1[r] = gf(row[a.a1_off + r]);
  for (int c = tid; c < a.dim; c += kGdThreads) {
    s_q[c] = gf(row[a.q_off + h * a.dim + c]) * a.q_scale;
    s_k[c] = gf(row[a.k_off + h * a.dim + c]);
  }
  __syncthreads();
  const T* a2 = static_cast<const T*>(a.a2) + static_cast<int64_t>(h) * a.dim * a.rank;
  for (int c = tid; c < a.dim; c += kGdThreads) {
    float z = a.a2_bias[h * a.dim + c];
    for (int r = 0; r < a.rank; ++r) z += s_a1[r] * gf(a2[c * a.rank + r]);
    s_al[c] = expf(log_sigmoid(z) * a.inv_tau);
  }
  __syncthreads();
  float* S = a.state + (static_cast<int64_t>(b) * a.heads + h) * a.dim * a.vdim;
  const int nc = (a.vdim + V - 1) / V;              // vector columns
  const int cols = min(nc, kGdThreads);             // columns handled side by side
  const int groups = kGdThreads / cols;             // rows handled side by side
  const int rg = tid / cols;
  for (int i = tid; i < groups * a.vdim; i += kGdThreads) s_o[i] = 0.f;
  __syncthreads();
  if (rg < groups) {
    for (int cv = tid % cols; cv < nc; cv += cols) {
      float v[V], o[V];
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = gf(row[a.v_off + h * a.vdim + cv * V + i]), o[i] = 0.f;
      float* p = S + cv * V;
#pragma unroll 4
      for (int c = rg; c < a.dim; c += groups) {
        const float al = s_al[c], k = s_k[c], q = s_q[c];
        float* e = p + static_cast<int64_t>(c) * a.vdim;
        if (V == 4) {
          float4 s = *reinterpret_cast<const float4*>(e);
          s.x = al * s.x + k * v[0], s.y = al * s.y + k * v[1 % V];
          s.z = al * s.z + k * v[2 % V], s.w = al * s.w + k * v[3 % V];
          *reinterpret_cast<float4*>(e) = s;
          o[0] += q * s.x, o[1 % V] += q * s.y, o[2 % V] += q * s.z, o[3 % V] += q * s.w;
        } else {
          const float s = al * e[0] + k * v[0];
          e[0] = s;
          o[0] += q * s;
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) s_o[rg * a.vdim + cv * V + i] = o[i];
    }
  }
  __syncthreads();
  float sq = 0.f;
  for (int d = tid; d < a.vdim; d += kGdThreads) {
    float o = 0.f;
    for (int g = 0; g < groups; ++g) o += s_o[g * a.vdim + d];
    s_o[d] = o;  // group 0's row; read above by this thread only
    sq += o * o;
  }
  for (int off = 16; off > 0; off >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, off);
  if ((tid & 31) == 0) s_red[tid >> 5] = sq;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (int w = 0; w < kGdThreads / 32; ++w) total += s_red[w];
  const float inv = rsqrtf(total / a.vdim + a.eps);
  for (int d = tid; d < a.vdim; d += kGdThreads)
    out[d] = T(s_o[d] * inv * a.norm_w[d] * silu(gf(row[a.g_off + h * a.vdim + d])));
}

constexpr int kGsTok = 16, kGsCols = 32, kGsThreads = 256;

// State slice [dim, 32] of one head in registers: thread (row group, column), RPT rows per thread.
template <typename T, int RPT>
__global__ void __launch_bounds__(kGsThreads) gla_scan_kernel(GlaArgs a) {
  extern __shared__ float sm[];
  const int h = blockIdx.y, b = blockIdx.z, d0 = blockIdx.x * kGsCols;
  const int tid = threadIdx.x, rg = tid / kGsCols, col = tid % kGsCols;
  constexpr int RG = kGsThreads / kGsCols;
  if (row_inactive(a, b)) return;  // the norm kernel writes zeros
  const int live = live_tokens(a, b);
  float* s_q = sm;                          // [16][dim]
  float* s_k = s_q + kGsTok * a.dim;
  float* s_al = s_k + kGsTok * a.dim;
  float* s_v = s_al + kGsTok * a.dim;       // [16][32]
  float* s_o = s_v + kGsTok * kGsCols;      // [16][RG][32]
  float* s_a1 = s_o + kGsTok * kGsThreads;  // [16][rank]
  const bool in = d0 + col < a.vdim;
  float* S = a.state + (static_cast<int64_t>(b) * a.heads + h) * a.dim * a.vdim + d0 + col;
  float st[RPT];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int c = rg + r * RG;
    st[r] = in && c < a.dim ? S[static_cast<int64_t>(c) * a.vdim] : 0.f;
  }
  const T* base = static_cast<const T*>(a.proj) + static_cast<int64_t>(b) * a.T * a.ld;
  const T* a2 = static_cast<const T*>(a.a2) + static_cast<int64_t>(h) * a.dim * a.rank;
  for (int t0 = 0; t0 < live; t0 += kGsTok) {
    const int n = min(kGsTok, live - t0);
    __syncthreads();
    for (int i = tid; i < n * a.rank; i += kGsThreads)
      s_a1[i] = gf(base[(t0 + i / a.rank) * a.ld + a.a1_off + i % a.rank]);
    for (int i = tid; i < n * kGsCols; i += kGsThreads) {
      const int d = d0 + i % kGsCols;
      s_v[i] = d < a.vdim ? gf(base[(t0 + i / kGsCols) * a.ld + a.v_off + h * a.vdim + d]) : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < n * a.dim; i += kGsThreads) {
      const int t = i / a.dim, c = i % a.dim;
      const T* row = base + (t0 + t) * a.ld;
      s_q[i] = gf(row[a.q_off + h * a.dim + c]) * a.q_scale;
      s_k[i] = gf(row[a.k_off + h * a.dim + c]);
      float z = a.a2_bias[h * a.dim + c];
      for (int r = 0; r < a.rank; ++r) z += s_a1[t * a.rank + r] * gf(a2[c * a.rank + r]);
      s_al[i] = expf(log_sigmoid(z) * a.inv_tau);
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float v = s_v[t * kGsCols + col];
      float o = 0.f;
#pragma unroll
      for (int r = 0; r < RPT; ++r) {
        const int c = rg + r * RG;
        if (c < a.dim) {
          st[r] = s_al[t * a.dim + c] * st[r] + s_k[t * a.dim + c] * v;
          o += s_q[t * a.dim + c] * st[r];
        }
      }
      s_o[(t * RG + rg) * kGsCols + col] = o;
    }
    __syncthreads();
    for (int i = tid; i < n * kGsCols; i += kGsThreads) {
      const int t = i / kGsCols, c = i % kGsCols;
      if (d0 + c >= a.vdim) continue;
      float o = 0.f;
#pragma unroll
      for (int g = 0; g < RG; ++g) o += s_o[(t * RG + g) * kGsCols + c];
      a.o_raw[((static_cast<int64_t>(b) * a.T + t0 + t) * a.heads + h) * a.vdim + d0 + c] = o;
    }
  }
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int c = rg + r * RG;
    if (in && c < a.dim) S[static_cast<int64_t>(c) * a.vdim] = st[r];
  }
}

// out = rms(o_raw) * norm_w * silu(gate), one warp per (token, head); zeros beyond the live tokens.
template <typename T>
__global__ void gla_norm_gate_kernel(GlaArgs a) {
  const int64_t item = static_cast<int64_t>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= static_cast<int64_t>(a.B) * a.T * a.heads) return;
  const int h = static_cast<int>(item % a.heads);
  const int64_t tok = item / a.heads;
  const int b = static_cast<int>(tok / a.T), t = static_cast<int>(tok % a.T);
  T* out = static_cast<T*>(a.out) + tok * a.out_ld + h * a.vdim;
  if (row_inactive(a, b) || t >= live_tokens(a, b)) {
    for (int d = lane; d < a.vdim; d += 32) out[d] = T(0.f);
    return;
  }
  const float* o = a.o_raw + item * a.vdim;
  const T* g = static_cast<const T*>(a.proj) + tok * a.ld + a.g_off + h * a.vdim;
  float sq = 0.f;
  for (int d = lane; d < a.vdim; d += 32) sq += o[d] * o[d];
  for (int off = 16; off > 0; off >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, off);
  const float inv = rsqrtf(sq / a.vdim + a.eps);
  for (int d = lane; d < a.vdim; d += 32) out[d] = T(o[d] * inv * a.norm_w[d] * silu(gf(g[d])));
}

// ------------------------------------------------------------------------------------------
// Chunked form on the tensor cores.
// ------------------------------------------------------------------------------------------
//
// Within a chunk of 64 tokens let G_i be the running sum of ld (inclusive), a vector over channels.
//   q^_i = q_i exp(G_i)      k~_j = k_j exp(-G_j)
//   o_i  = S_in^T q^_i + sum_{j <= i} (q^_i . k~_j) v_j
//   S_out = diag(exp(G_64)) (S_in + sum_j k~_j v_j^T)
// (the code keeps G in base 2).
// The factored form is exact as long as exp(-G_64) stays finite: a chunk with a channel whose total
// decay exceeds 2^-86 is run token by token on the same register state instead (a uniform branch).
//
// What enters the recurrence is kept to fp32 accuracy: k~, the scores and the state as matrix operands
// are split into two bf16 terms (hi + lo); q^ is one bf16, like the projection q itself.
//
// One CTA = 8 warps per (64 or 128 value columns, head, sequence, segment of the prompt).  Warp w owns
// VS / 8 value columns of the state, held transposed as mma accumulators (rows = value columns, columns =
// key channels): in that layout the accumulator registers ARE the B fragments of S_in^T q^.  Projections,
// decays and scores are shared through shared memory; two CTAs share an SM and overlap each other.
//
// Long prompts of few sequences are cut into segments: a first launch (kStateOnly) computes what each
// segment alone adds to the state and its total decay, gla_segment_kernel chains them, and the second
// launch runs every segment from its true initial state.
namespace {

constexpr int kGcTok = 64, kGcThreads = 256;

__device__ __forceinline__ void prefetch_row(const __nv_bfloat16* p, int n) {
  for (int c = 0; c < n; c += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(p + c));
}

// 64 rows of `n` elements (source pitch ld) into a tile of W columns, zero beyond n and beyond `rows`.  A
// thread keeps its column and walks the rows.
template <int W>
__device__ __forceinline__ void load_tile(__nv_bfloat16* tile, int pitch, const __nv_bfloat16* src, int64_t ld, int n,
                                          int rows, bool vec) {
  constexpr int kPer = W / 8, kStep = kGcThreads / kPer;
  const int c = (threadIdx.x % kPer) * 8, r0 = threadIdx.x / kPer;
  __nv_bfloat16* dst = tile + r0 * pitch + c;
  const __nv_bfloat16* p = src + r0 * ld + c;
  const bool whole = vec && c + 8 <= n;
#pragma unroll
  for (int r = r0; r < kGcTok; r += kStep) {
    if (whole && r < rows) {
      cp16(dst, p);
    } else if (vec || c >= n || r >= rows) {
      *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    } else {
#pragma unroll 1
      for (int e = 0; e < 8; ++e) dst[e] = c + e < n ? p[e] : __float2bfloat16(0.f);
    }
    dst += kStep * pitch;
    p += kStep * ld;
  }
}

__device__ __forceinline__ float lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float kLog2e = 1.4426950408889634f;
// x * sigmoid(x)
__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.f + ex2(-x * kLog2e)); }

}  // namespace

template <int DP, int VS>
struct GcSmem {
  static constexpr int kQP = DP + 8, kVP = VS + 8, kAP = kGcTok + 8;
  static constexpr int kQ = 0;                               // bf16 [64][kQP]  q, then q^; [64][kVP] gate, then out
  static constexpr int kK = kQ + kGcTok * (kQP > kVP ? kQP : kVP) * 2;  // bf16 k, then k~ hi
  static constexpr int kV = kK + kGcTok * kQP * 2;           // bf16 [64][kVP]
  static constexpr int kKlo = kV + kGcTok * kVP * 2;         // bf16 [64][kQP]  k~ lo   } token-by-token path:
  static constexpr int kA = kKlo + kGcTok * kQP * 2;         // bf16 2 x [64][kAP]      } fp32 decay [64][DP]
  static constexpr int kEnd = kA + 2 * kGcTok * kAP * 2;     // float [DP]  exp(G_64)
  static constexpr int kSum = kEnd + DP * 4;                 // float [DP]  total log decay of the segment
  static constexpr int kRow = kSum + DP * 4;                 // float [64][8] row sums of squares
  static constexpr int kBias = kRow + kGcTok * 8 * 4;        // float [DP]
  static constexpr int kA2 = kBias + DP * 4;                 // bf16 [DP][rp + 8], then a1 bf16 [64][rp + 8]
  static_assert(kGcTok * kQP * 2 + 2 * kGcTok * kAP * 2 >= kGcTok * DP * 4, "decay overlay");
  static size_t total(int rp) { return kA2 + static_cast<size_t>(DP + kGcTok) * (rp + 8) * 2; }
};

template <int DP, int VS, bool kStateOnly>
__global__ void __launch_bounds__(kGcThreads, 2) gla_chunk_kernel(GlaArgs a) {
  using L = GcSmem<DP, VS>;
  using bf16 = __nv_bfloat16;
  constexpr int MV = VS / 128 > 0 ? VS / 128 : 1;  // 16-row state tiles per warp
  constexpr int kWarpsV = VS / (16 * MV);          // warps that own value columns
  constexpr int NT = DP / 8;                       // 8-channel state tiles
  constexpr int ZT = DP / 64;                      // 8-channel decay tiles per warp
  extern __shared__ __align__(16) uint8_t gla_smem[];
  bf16* sQ = reinterpret_cast<bf16*>(gla_smem + L::kQ);
  bf16* sK = reinterpret_cast<bf16*>(gla_smem + L::kK);
  bf16* sV = reinterpret_cast<bf16*>(gla_smem + L::kV);
  bf16* sKlo = reinterpret_cast<bf16*>(gla_smem + L::kKlo);
  bf16* sAhi = reinterpret_cast<bf16*>(gla_smem + L::kA);
  bf16* sAlo = sAhi + kGcTok * L::kAP;
  float* sDecay = reinterpret_cast<float*>(gla_smem + L::kKlo);
  float* sEnd = reinterpret_cast<float*>(gla_smem + L::kEnd);
  float* sSum = reinterpret_cast<float*>(gla_smem + L::kSum);
  float* sRow = reinterpret_cast<float*>(gla_smem + L::kRow);
  float* sBias = reinterpret_cast<float*>(gla_smem + L::kBias);
  const int rp = (a.rank + 15) / 16 * 16, rpp = rp + 8;
  bf16* sA2 = reinterpret_cast<bf16*>(gla_smem + L::kA2);
  bf16* sA1 = sA2 + DP * rpp;

  const int slices = (a.vdim + VS - 1) / VS;
  const int seg = blockIdx.x / slices, d0 = (blockIdx.x % slices) * VS;
  const int h = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lc = (lane & 3) * 2;
  const bool inactive = row_inactive(a, b);
  const int live = inactive ? 0 : live_tokens(a, b);
  const int t_lo = seg * a.seg_tokens, t_hi = a.segments > 1 ? min(a.T, t_lo + a.seg_tokens) : a.T;
  const int vcols = min(VS, a.vdim - d0);
  const bf16* base = static_cast<const bf16*>(a.proj) + static_cast<int64_t>(b) * a.T * a.ld;
  const bool vec = !((a.ld | a.q_off | a.k_off | a.v_off | a.g_off | a.dim | a.vdim) & 7);
  const bool vec_a1 = vec && !((a.a1_off | a.rank) & 7);
  const bool owner = warp < kWarpsV;
  const int v0 = warp * 16 * MV;  // first value column of this warp in the slice
  const float mean_scale = a.q_scale * a.q_scale / a.vdim;  // outputs are scaled by q_scale at the end
  float nw[MV * 2][2];
#pragma unroll
  for (int n = 0; n < MV * 2; ++n)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int v = v0 + n * 8 + lc + e;
      nw[n][e] = !kStateOnly && slices == 1 && owner && v < vcols ? a.norm_w[v] : 0.f;
    }

  for (int i = tid; i < DP * rp; i += kGcThreads) {
    const int c = i / rp, r = i % rp;
    sA2[c * rpp + r] = c < a.dim && r < a.rank
                           ? static_cast<const bf16*>(a.a2)[(static_cast<int64_t>(h) * a.dim + c) * a.rank + r]
                           : __float2bfloat16(0.f);
  }
  for (int c = tid; c < DP; c += kGcThreads) {
    sBias[c] = c < a.dim ? a.a2_bias[h * a.dim + c] * kLog2e : 0.f;
    sSum[c] = 0.f;
  }

  // State, transposed: row = value column, column = key channel.
  float S[MV][NT][4];
  const bool segmented = a.segments > 1;
  float* state = a.state + (static_cast<int64_t>(b) * a.heads + h) * a.dim * a.vdim;
  float* seg_state = segmented
                         ? a.seg_state + ((static_cast<int64_t>(b) * a.heads + h) * a.segments + seg) * a.dim * a.vdim
                         : nullptr;
  const float* init = segmented ? seg_state : state;
#pragma unroll
  for (int mv = 0; mv < MV; ++mv)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int v = v0 + mv * 16 + lr + (e >> 1) * 8, c = n * 8 + lc + (e & 1);
        S[mv][n][e] = !kStateOnly && owner && v < vcols && c < a.dim ? init[static_cast<int64_t>(c) * a.vdim + d0 + v] : 0.f;
      }

  for (int t0 = t_lo; t0 < t_hi; t0 += kGcTok) {
    const int rows = max(0, min(kGcTok, min(live, t_hi) - t0));
    if (rows == 0) {
      // Nothing live here or later in this segment: zero the outputs.
      if (!kStateOnly) {
        const int n = min(kGcTok, t_hi - t0);
        for (int i = tid; i < n * vcols; i += kGcThreads) {
          const int64_t tok = static_cast<int64_t>(b) * a.T + t0 + i / vcols;
          if (slices == 1)
            static_cast<bf16*>(a.out)[tok * a.out_ld + h * a.vdim + i % vcols] = __float2bfloat16(0.f);
        }
      }
      continue;
    }
    __syncthreads();  // everybody is done with the previous chunk's tiles
    const bf16* src = base + static_cast<int64_t>(t0) * a.ld;
    if (!kStateOnly) load_tile<DP>(sQ, L::kQP, src + a.q_off + h * a.dim, a.ld, a.dim, rows, vec);
    load_tile<DP>(sK, L::kQP, src + a.k_off + h * a.dim, a.ld, a.dim, rows, vec);
    load_tile<VS>(sV, L::kVP, src + a.v_off + h * a.vdim + d0, a.ld, vcols, rows, vec);
    if (vec_a1) {
      for (int i = tid; i < kGcTok * (rp / 8); i += kGcThreads) {
        const int r = i / (rp / 8), c = (i % (rp / 8)) * 8;
        if (r < rows && c < a.rank)
          cp16(sA1 + r * rpp + c, src + r * a.ld + a.a1_off + c);
        else
          *reinterpret_cast<uint4*>(sA1 + r * rpp + c) = make_uint4(0, 0, 0, 0);
      }
    } else {
      for (int i = tid; i < kGcTok * rp; i += kGcThreads) {
        const int r = i / rp, c = i % rp;
        sA1[r * rpp + c] = r < rows && c < a.rank ? src[r * a.ld + a.a1_off + c] : __float2bfloat16(0.f);
      }
    }
    // The next chunk's rows start their way from DRAM to L2 while this one is computed.
    if (t0 + kGcTok + (tid >> 2) < min(live, t_hi)) {
      const bf16* next = src + (kGcTok + (tid >> 2)) * a.ld;
      switch (tid & 3) {
        case 0: prefetch_row(next + a.q_off + h * a.dim, kStateOnly ? 0 : a.dim); break;
        case 1: prefetch_row(next + a.k_off + h * a.dim, a.dim); break;
        case 2: prefetch_row(next + a.v_off + h * a.vdim + d0, vcols); break;
        default: prefetch_row(next + a.g_off + h * a.vdim + d0, kStateOnly ? 0 : vcols); break;
      }
    }
    cp_wait_all();
    __syncthreads();
    auto load_gate = [&]() {  // over q^, once nobody reads it any more
      if (!kStateOnly && slices == 1) load_tile<VS>(sQ, L::kVP, src + a.g_off + h * a.vdim, a.ld, vcols, rows, vec);
    };

    // Log decays of this warp's channels [warp * DP / 8, + DP / 8): rows = tokens.
    float g[4][ZT][4];
    auto log_decays = [&]() {
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int n = 0; n < ZT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) g[m][n][e] = 0.f;
      for (int k0 = 0; k0 < rp; k0 += 16) {
        uint32_t bfr[ZT][2];
#pragma unroll
        for (int n = 0; n < ZT; ++n) {
          const bf16* p = sA2 + (warp * (DP / 8) + n * 8 + lr) * rpp + k0 + lc;
          bfr[n][0] = *reinterpret_cast<const uint32_t*>(p);
          bfr[n][1] = *reinterpret_cast<const uint32_t*>(p + 8);
        }
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          uint32_t afr[4];
          ldsm4(afr, sA1 + (m * 16 + (lane & 15)) * rpp + k0 + (lane >> 4) * 8);
#pragma unroll
          for (int n = 0; n < ZT; ++n) mma(g[m][n], afr, bfr[n][0], bfr[n][1]);
        }
      }
#pragma unroll
      for (int n = 0; n < ZT; ++n) {
        // In base 2: log2 sigmoid(z) = min(z', 0) - log2(1 + 2^-|z'|), z' = z log2(e).
        const int c = warp * (DP / 8) + n * 8 + lc;
        const float2 bias = *reinterpret_cast<const float2*>(sBias + c);
        const float t0 = c < a.dim ? a.inv_tau : 0.f, t1 = c + 1 < a.dim ? a.inv_tau : 0.f;
#pragma unroll
        for (int m = 0; m < 4; ++m)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float z = fmaf(g[m][n][e], kLog2e, e & 1 ? bias.y : bias.x);
            g[m][n][e] = (fminf(z, 0.f) - lg2(1.f + ex2(-fabsf(z)))) * (e & 1 ? t1 : t0);
          }
        if (rows < kGcTok) {
#pragma unroll
          for (int m = 0; m < 4; ++m)
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (m * 16 + lr + (e >> 1) * 8 >= rows) g[m][n][e] = 0.f;
        }
      }
    };
    log_decays();
    // Running sums over the 64 tokens: lanes with equal lane & 3 hold rows lr, lr + 8, ...
    float worst = 0.f;
    float g_end[ZT][2];
#pragma unroll
    for (int n = 0; n < ZT; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float carry = 0.f;
#pragma unroll
        for (int blk = 0; blk < 8; ++blk) {
          float x = g[blk >> 1][n][(blk & 1) * 2 + e];
#pragma unroll
          for (int off = 4; off <= 16; off <<= 1) {
            const float y = __shfl_up_sync(0xffffffffu, x, off);
            if (lane >= off) x += y;
          }
          x += carry;
          carry = __shfl_sync(0xffffffffu, x, 28 + (lane & 3));
          g[blk >> 1][n][(blk & 1) * 2 + e] = x;
        }
        g_end[n][e] = carry;
        worst = fminf(worst, carry);
      }
    const bool sequential = __syncthreads_or(worst < -86.f);
    if (lr == 0) {
#pragma unroll
      for (int n = 0; n < ZT; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int c = warp * (DP / 8) + n * 8 + lc + e;
          sEnd[c] = ex2(g_end[n][e]);
          if (kStateOnly) sSum[c] += g_end[n][e];
        }
    }

    float O[4][MV * 2][4];
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
      for (int n = 0; n < MV * 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) O[m][n][e] = 0.f;

    if (!sequential) {
      // q^ and k~ in place; every element is touched by the thread that owns its decay.
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int n = 0; n < ZT; ++n)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int r = m * 16 + lr + half * 8, c = warp * (DP / 8) + n * 8 + lc;
            const float g0 = g[m][n][half * 2], g1 = g[m][n][half * 2 + 1];
            if (!kStateOnly) {
              uint32_t* pq = reinterpret_cast<uint32_t*>(sQ + r * L::kQP + c);
              const float2 q = unpack2(*pq);
              *pq = pack2(q.x * ex2(g0), q.y * ex2(g1));
            }
            uint32_t* pk = reinterpret_cast<uint32_t*>(sK + r * L::kQP + c);
            const float2 k = unpack2(*pk);
            uint32_t hi, lo;
            split2(k.x * ex2(-g0), k.y * ex2(-g1), hi, lo);
            *pk = hi;
            *reinterpret_cast<uint32_t*>(sKlo + r * L::kQP + c) = lo;
          }
      __syncthreads();

      if (!kStateOnly) {
        // Scores: warp w computes rows [16 (w & 3), + 16), keys [32 (w >> 2), + 32).
        const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 32;
        float A[4][4];
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) A[n][e] = 0.f;
        if (n0 <= m0 + 15) {
#pragma unroll
          for (int k0 = 0; k0 < DP; k0 += 16) {
            uint32_t af[4];
            ldsm4(af, sQ + (m0 + (lane & 15)) * L::kQP + k0 + (lane >> 4) * 8);
#pragma unroll
            for (int p = 0; p < 2; ++p) {
              if (n0 + p * 16 <= m0 + 15) {
                uint32_t bh[4], bl[4];
                const int off = (n0 + p * 16 + (lane >> 4) * 8 + (lane & 7)) * L::kQP + k0 + ((lane >> 3) & 1) * 8;
                ldsm4(bh, sK + off);
                ldsm4(bl, sKlo + off);
                mma(A[2 * p], af, bh[0], bh[1]);
                mma(A[2 * p + 1], af, bh[2], bh[3]);
                mma(A[2 * p], af, bl[0], bl[1]);
                mma(A[2 * p + 1], af, bl[2], bl[3]);
              }
            }
          }
        }
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int r = m0 + lr + half * 8, c = n0 + n * 8 + lc;
            uint32_t hi, lo;
            split2(c <= r ? A[n][half * 2] : 0.f, c + 1 <= r ? A[n][half * 2 + 1] : 0.f, hi, lo);
            *reinterpret_cast<uint32_t*>(sAhi + r * L::kAP + c) = hi;
            *reinterpret_cast<uint32_t*>(sAlo + r * L::kAP + c) = lo;
          }
        if (owner) {
          // O += q^ S_in: the state's accumulators as B fragments, hi and lo.
#pragma unroll
          for (int kk = 0; kk < DP / 16; ++kk) {
            uint32_t bh[MV * 2][2], bl[MV * 2][2];
#pragma unroll
            for (int mv = 0; mv < MV; ++mv)
#pragma unroll
              for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int t = 0; t < 2; ++t)
                  split2(S[mv][2 * kk + t][2 * u], S[mv][2 * kk + t][2 * u + 1], bh[mv * 2 + u][t], bl[mv * 2 + u][t]);
#pragma unroll
            for (int m = 0; m < 4; ++m) {
              uint32_t af[4];
              ldsm4(af, sQ + (m * 16 + (lane & 15)) * L::kQP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
              for (int n = 0; n < MV * 2; ++n) {
                mma(O[m][n], af, bh[n][0], bh[n][1]);
                mma(O[m][n], af, bl[n][0], bl[n][1]);
              }
            }
          }
        }
        __syncthreads();
        load_gate();
        if (owner) {
          // O += A V.
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) {
            uint32_t bv[MV][4];
#pragma unroll
            for (int mv = 0; mv < MV; ++mv)
              ldsm4t(bv[mv], sV + (kk * 16 + (lane & 15)) * L::kVP + v0 + mv * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int m = kk; m < 4; ++m) {
              uint32_t ah[4], al[4];
              const int off = (m * 16 + (lane & 15)) * L::kAP + kk * 16 + (lane >> 4) * 8;
              ldsm4(ah, sAhi + off);
              ldsm4(al, sAlo + off);
#pragma unroll
              for (int mv = 0; mv < MV; ++mv)
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                  mma(O[m][mv * 2 + u], ah, bv[mv][2 * u], bv[mv][2 * u + 1]);
                  mma(O[m][mv * 2 + u], al, bv[mv][2 * u], bv[mv][2 * u + 1]);
                }
            }
          }
        }
      }
      if (owner) {
        // S += V^T k~ (hi and lo), then the chunk's total decay per channel.
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          uint32_t av[MV][4];
#pragma unroll
          for (int mv = 0; mv < MV; ++mv)
            ldsm4t(av[mv], sV + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * L::kVP + v0 + mv * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
          for (int n = 0; n < NT; n += 2) {
            uint32_t bh[4], bl[4];
            const int off = (kk * 16 + (lane & 15)) * L::kQP + n * 8 + (lane >> 4) * 8;
            ldsm4t(bh, sK + off);
            ldsm4t(bl, sKlo + off);
#pragma unroll
            for (int mv = 0; mv < MV; ++mv) {
              mma(S[mv][n], av[mv], bh[0], bh[1]);
              mma(S[mv][n + 1], av[mv], bh[2], bh[3]);
              mma(S[mv][n], av[mv], bl[0], bl[1]);
              mma(S[mv][n + 1], av[mv], bl[2], bl[3]);
            }
          }
        }
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const float2 d = *reinterpret_cast<const float2*>(sEnd + n * 8 + lc);
#pragma unroll
          for (int mv = 0; mv < MV; ++mv) S[mv][n][0] *= d.x, S[mv][n][1] *= d.y, S[mv][n][2] *= d.x, S[mv][n][3] *= d.y;
        }
      }
    } else {
      // Token by token: decays as such, state and outputs in fp32.
      log_decays();
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int n = 0; n < ZT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            sDecay[(m * 16 + lr + (e >> 1) * 8) * DP + warp * (DP / 8) + n * 8 + lc + (e & 1)] = exp2f(g[m][n][e]);
      __syncthreads();
      if (owner) {
        for (int t = 0; t < rows; ++t) {
          float v[MV][2], o[MV][2];
#pragma unroll
          for (int mv = 0; mv < MV; ++mv)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              v[mv][u] = __bfloat162float(sV[t * L::kVP + v0 + mv * 16 + lr + u * 8]);
              o[mv][u] = 0.f;
            }
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            const int c = n * 8 + lc;
            const float2 al = *reinterpret_cast<const float2*>(sDecay + t * DP + c);
            const float2 k = unpack2(*reinterpret_cast<const uint32_t*>(sK + t * L::kQP + c));
            float2 q = make_float2(0.f, 0.f);
            if (!kStateOnly) q = unpack2(*reinterpret_cast<const uint32_t*>(sQ + t * L::kQP + c));
#pragma unroll
            for (int mv = 0; mv < MV; ++mv)
#pragma unroll
              for (int u = 0; u < 2; ++u) {
                float& s0 = S[mv][n][2 * u];
                float& s1 = S[mv][n][2 * u + 1];
                s0 = al.x * s0 + k.x * v[mv][u];
                s1 = al.y * s1 + k.y * v[mv][u];
                o[mv][u] += q.x * s0 + q.y * s1;
              }
          }
          if (!kStateOnly) {
#pragma unroll
            for (int mv = 0; mv < MV; ++mv)
#pragma unroll
              for (int u = 0; u < 2; ++u) {
                float x = o[mv][u];
                x += __shfl_xor_sync(0xffffffffu, x, 1);
                x += __shfl_xor_sync(0xffffffffu, x, 2);
                // Lane (lr, *) now holds token t, column lr + 8 u; an O fragment wants row t at lanes with
                // lr == t % 8, columns 2 (lane & 3), + 1.
                const float y0 = __shfl_sync(0xffffffffu, x, lc * 4), y1 = __shfl_sync(0xffffffffu, x, (lc + 1) * 4);
                if (lr == (t & 7)) {
#pragma unroll
                  for (int m = 0; m < 4; ++m)
#pragma unroll
                    for (int half = 0; half < 2; ++half)
                      if (t >> 3 == m * 2 + half) {
                        O[m][mv * 2 + u][half * 2] = y0;
                        O[m][mv * 2 + u][half * 2 + 1] = y1;
                      }
                }
              }
          }
        }
      }
      __syncthreads();
      load_gate();
    }
    if (kStateOnly) continue;

    // Outputs.
    if (slices > 1) {
      if (owner) {
#pragma unroll
        for (int m = 0; m < 4; ++m)
#pragma unroll
          for (int n = 0; n < MV * 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int r = m * 16 + lr + (e >> 1) * 8, v = v0 + n * 8 + lc + (e & 1);
              if (r < rows && v < vcols)
                a.o_raw[((static_cast<int64_t>(b) * a.T + t0 + r) * a.heads + h) * a.vdim + d0 + v] = O[m][n][e] * a.q_scale;
            }
      }
      continue;
    }
    if (owner) {
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          float sq = 0.f;
#pragma unroll
          for (int n = 0; n < MV * 2; ++n)
            sq += O[m][n][half * 2] * O[m][n][half * 2] + O[m][n][half * 2 + 1] * O[m][n][half * 2 + 1];
          sq += __shfl_xor_sync(0xffffffffu, sq, 1);
          sq += __shfl_xor_sync(0xffffffffu, sq, 2);
          if ((lane & 3) == 0) sRow[(m * 16 + lr + half * 8) * 8 + warp] = sq;
        }
    }
    cp_wait_all();
    __syncthreads();
    if (owner) {
      // Dead rows have zero outputs and gates.
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = m * 16 + lr + half * 8;
          const float4 s0 = *reinterpret_cast<const float4*>(sRow + r * 8);
          float total = s0.x + s0.y + s0.z + s0.w;
          if (kWarpsV > 4) {
            const float4 s1 = *reinterpret_cast<const float4*>(sRow + r * 8 + 4);
            total += s1.x + s1.y + s1.z + s1.w;
          }
          const float inv = a.q_scale * rsqrtf(total * mean_scale + a.eps);
#pragma unroll
          for (int n = 0; n < MV * 2; ++n) {
            uint32_t* p = reinterpret_cast<uint32_t*>(sQ + r * L::kVP + v0 + n * 8 + lc);
            const float2 x = unpack2(*p);
            *p = pack2(O[m][n][half * 2] * inv * nw[n][0] * silu_fast(x.x),
                       O[m][n][half * 2 + 1] * inv * nw[n][1] * silu_fast(x.y));
          }
        }
    }
    __syncthreads();
    const int n_out = min(kGcTok, t_hi - t0);
    bf16* out = static_cast<bf16*>(a.out) + (static_cast<int64_t>(b) * a.T + t0) * a.out_ld + h * a.vdim;
    if (vec) {
      const int c = (tid % (VS / 8)) * 8;
      bf16* p = out + (tid / (VS / 8)) * a.out_ld + c;
#pragma unroll
      for (int r = tid / (VS / 8); r < kGcTok; r += kGcThreads / (VS / 8)) {
        if (r < n_out && c < vcols) *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(sQ + r * L::kVP + c);
        p += kGcThreads / (VS / 8) * a.out_ld;
      }
    } else {
      for (int i = tid; i < n_out * vcols; i += kGcThreads) {
        const int r = i / vcols, c = i % vcols;
        out[r * a.out_ld + c] = sQ[r * L::kVP + c];
      }
    }
  }

  // Final state: of the sequence (last segment), or of this segment alone.
  if (!kStateOnly && (segmented ? seg != a.segments - 1 : false)) return;
  if (inactive && !kStateOnly) return;
  float* dst = kStateOnly ? seg_state : state;
#pragma unroll
  for (int mv = 0; mv < MV; ++mv)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int v = v0 + mv * 16 + lr + (e >> 1) * 8, c = n * 8 + lc + (e & 1);
        if (owner && v < vcols && c < a.dim) dst[static_cast<int64_t>(c) * a.vdim + d0 + v] = S[mv][n][e];
      }
  if (kStateOnly && d0 == 0) {
    __syncthreads();
    for (int c = tid; c < a.dim; c += kGcThreads)
      a.seg_decay[((static_cast<int64_t>(b) * a.heads + h) * a.segments + seg) * a.dim + c] = sSum[c];
  }
}

// Chains the segments: on entry seg_state[s] is what segment s adds to a zero state, on exit the state
// at the segment's start.
__global__ void gla_segment_kernel(GlaArgs a) {
  const int64_t bh = blockIdx.y;
  const int64_t n = static_cast<int64_t>(a.dim) * a.vdim;
  const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int c = static_cast<int>(i / a.vdim);
  float s = a.state[bh * n + i];
  for (int g = 0; g < a.segments; ++g) {
    float* p = a.seg_state + (bh * a.segments + g) * n + i;
    const float add = *p;
    *p = s;
    s = s * exp2f(a.seg_decay[(bh * a.segments + g) * a.dim + c]) + add;
  }
}

namespace {

template <typename T>
int norm_gate(const GlaArgs& a, cudaStream_t stream) {
  const int64_t items = static_cast<int64_t>(a.B) * a.T * a.heads;
  gla_norm_gate_kernel<T><<<static_cast<unsigned>((items + 7) / 8), 256, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename T, int RPT>
int launch_scan(const GlaArgs& a, cudaStream_t stream) {
  const size_t smem = sizeof(float) * (3 * kGsTok * a.dim + kGsTok * kGsCols + kGsTok * kGsThreads + kGsTok * a.rank);
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    if (smem > 220 * 1024 || cudaFuncSetAttribute(gla_scan_kernel<T, RPT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                  static_cast<int>(smem)) != cudaSuccess)
      return -3;
    configured = smem;
  }
  const dim3 grid((a.vdim + kGsCols - 1) / kGsCols, a.heads, a.B);
  gla_scan_kernel<T, RPT><<<grid, kGsThreads, smem, stream>>>(a);
  if (cudaGetLastError() != cudaSuccess) return -4;
  return norm_gate<T>(a, stream);
}

template <typename T>
int scan(const GlaArgs& a, cudaStream_t stream) {
  if (a.dim <= 64) return launch_scan<T, 8>(a, stream);
  if (a.dim <= 128) return launch_scan<T, 16>(a, stream);
  if (a.dim <= 256) return launch_scan<T, 32>(a, stream);
  return launch_scan<T, 64>(a, stream);
}

template <typename T, int V>
int launch_gla_decode(const GlaArgs& a, cudaStream_t stream) {
  const int nc = (a.vdim + V - 1) / V;
  const int groups = kGdThreads / (nc < kGdThreads ? nc : kGdThreads);
  const size_t smem = sizeof(float) * (3 * a.dim + (a.rank + 3) / 4 * 4 + static_cast<size_t>(groups) * a.vdim);
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    if (smem > 220 * 1024 || cudaFuncSetAttribute(gla_decode_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                  static_cast<int>(smem)) != cudaSuccess)
      return -3;
    configured = smem;
  }
  gla_decode_kernel<T, V><<<dim3(a.heads, a.B), kGdThreads, smem, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <int DP, int VS, bool kStateOnly>
int launch_chunk_pass(const GlaArgs& a, cudaStream_t stream) {
  const int rp = (a.rank + 15) / 16 * 16;
  const size_t smem = GcSmem<DP, VS>::total(rp);
  auto kernel = gla_chunk_kernel<DP, VS, kStateOnly>;
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    if (smem > 220 * 1024 || cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                  static_cast<int>(smem)) != cudaSuccess)
      return -3;
    configured = smem;
  }
  const int slices = (a.vdim + VS - 1) / VS;
  kernel<<<dim3(slices * a.segments, a.heads, a.B), kGcThreads, smem, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <int DP, int VS>
int launch_chunk(const GlaArgs& a, cudaStream_t stream) {
  if (a.segments > 1) {
    int rc = launch_chunk_pass<DP, VS, true>(a, stream);
    if (rc) return rc;
    const int64_t n = static_cast<int64_t>(a.dim) * a.vdim;
    gla_segment_kernel<<<dim3(static_cast<unsigned>((n + 255) / 256), a.B * a.heads), 256, 0, stream>>>(a);
    if (cudaGetLastError() != cudaSuccess) return -4;
  }
  const int rc = launch_chunk_pass<DP, VS, false>(a, stream);
  if (rc || a.vdim <= VS) return rc;
  return norm_gate<__nv_bfloat16>(a, stream);
}

bool gla_bad(const GlaArgs& a) {
  return a.B <= 0 || a.T <= 0 || a.heads <= 0 || a.dim <= 0 || a.dim > 512 || a.vdim <= 0 || a.rank <= 0 ||
         a.rank > 512 || a.B > 65535 || a.heads > 65535 || a.out_ld < static_cast<int64_t>(a.heads) * a.vdim;
}

template <typename T>
__global__ void gla_zero_tail_kernel(T* out, int64_t rows, int64_t ld, int first) {
  const int pad = static_cast<int>(ld) - first;
  const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i < rows * pad) out[(i / pad) * ld + first + i % pad] = T(0.f);
}

int gla_zero_tail(const GlaArgs& a, cudaStream_t stream) {
  const int used = a.heads * a.vdim;
  if (a.out_ld == used) return 0;
  const int64_t rows = static_cast<int64_t>(a.B) * a.T, n = rows * (a.out_ld - used);
  const unsigned grid = static_cast<unsigned>((n + 255) / 256);
  if (a.act_bf16)
    gla_zero_tail_kernel<<<grid, 256, 0, stream>>>(static_cast<__nv_bfloat16*>(a.out), rows, a.out_ld, used);
  else
    gla_zero_tail_kernel<<<grid, 256, 0, stream>>>(static_cast<float*>(a.out), rows, a.out_ld, used);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace
}  // namespace axb

extern "C" int axb_gla_decode(const axb::GlaArgs* args, cudaStream_t stream) {
  const axb::GlaArgs& a = *args;
  if (axb::gla_bad(a) || a.T != 1) return -10;
  int rc;
  if (a.act_bf16)
    rc = a.vdim % 4 == 0 ? axb::launch_gla_decode<__nv_bfloat16, 4>(a, stream)
                         : axb::launch_gla_decode<__nv_bfloat16, 1>(a, stream);
  else
    rc = a.vdim % 4 == 0 ? axb::launch_gla_decode<float, 4>(a, stream) : axb::launch_gla_decode<float, 1>(a, stream);
  return rc ? rc : axb::gla_zero_tail(a, stream);
}

extern "C" int axb_gla_scan(const axb::GlaArgs* args, cudaStream_t stream) {
  const axb::GlaArgs& a = *args;
  if (axb::gla_bad(a) || a.o_raw == nullptr) return -10;
  const int rc = a.act_bf16 ? axb::scan<__nv_bfloat16>(a, stream) : axb::scan<float>(a, stream);
  return rc ? rc : axb::gla_zero_tail(a, stream);
}

// bf16 only; dim <= 128, rank <= 128.  segments > 1 needs seg_state / seg_decay and seg_tokens a
// multiple of 64 with segments * seg_tokens >= T; vdim > 128 needs o_raw.
extern "C" int axb_gla_chunk(const axb::GlaArgs* args, cudaStream_t stream) {
  const axb::GlaArgs& a = *args;
  if (axb::gla_bad(a) || !a.act_bf16 || a.dim > 128 || a.rank > 128 || a.segments < 1) return -10;
  if (a.segments > 1 && (a.seg_state == nullptr || a.seg_decay == nullptr || a.seg_tokens % 64 ||
                         static_cast<int64_t>(a.segments) * a.seg_tokens < a.T))
    return -11;
  if (a.vdim > 128 && a.o_raw == nullptr) return -11;
  int rc;
  if (a.dim <= 64)
    rc = a.vdim <= 64 ? axb::launch_chunk<64, 64>(a, stream) : axb::launch_chunk<64, 128>(a, stream);
  else
    rc = a.vdim <= 64 ? axb::launch_chunk<128, 64>(a, stream) : axb::launch_chunk<128, 128>(a, stream);
  return rc ? rc : axb::gla_zero_tail(a, stream);
}
