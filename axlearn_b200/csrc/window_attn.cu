// Gated sliding-window attention over a packed projection and a ring cache.
//
// The projections of a token lie in one row of `proj` ([B, T, ld]; q, k, v and the output gate at
// element offsets).  A sequence's last keys and values are kept in a ring of `slots` rows (position p in
// slot p % slots, layout [B, slots, G, dim]).  For query position i and key position j
//
//   score = (q . k) * scale * temp(i) - slope_h * (i - j),       0 <= i - j < window
//   temp(i) = 1 + coef * ln(floor((i + 1) / every) + 1)          (coef = 0: no temperature)
//   slope_h = 2^(-8 (h + 1) / H)                                 (bias = 0: none)
//   out     = softmax(score) V * sigmoid(gate)
//
// `start[b]` is the number of tokens the sequence already has in the ring (null: zero), `live[b]` the
// number of valid new tokens (null: T).  Three kernels:
//   window_decode_kernel  one new token per sequence; reads every visible key and value once, appends
//                         the new ones to the ring, splits long windows over CTAs (the last CTA to
//                         finish merges), applies the gate.
//   window_attn_kernel    any number of new tokens, any head sizes, fp32 or bf16: keys before `start`
//                         from the ring, the others from `proj` (fp32 runs, continued prompts, head
//                         sizes that the tensor-core kernel in flash_fwd_v3.cu does not take).
//   window_append_kernel  stores the last `slots` live tokens of a block of new tokens into the ring.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

namespace axb {

struct WindowArgs {
  const void* proj;
  void* k_ring;
  void* v_ring;
  void* out;             // [B, T, out_ld]
  const int* start;
  const int* live;
  float* part;           // decode splits: [B, H, splits, vdim + 2]
  int* tickets;          // [B * CTA groups], zero on entry and on exit
  int64_t ld, out_ld;
  int B, T, heads, kv_heads, dim, vdim, slots, window;
  int q_off, k_off, v_off, g_off;  // g_off < 0: no gate
  int splits, every, bias, act_bf16;
  float scale, coef;
};

namespace {

__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(__nv_bfloat16 x) { return __bfloat162float(x); }

__device__ __forceinline__ float query_scale(const WindowArgs& a, int pos) {
  if (a.coef == 0.f) return a.scale;
  return a.scale * (1.f + a.coef * logf(static_cast<float>((pos + 1) / a.every) + 1.f));
}
__device__ __forceinline__ float head_slope(const WindowArgs& a, int h) {
  return a.bias ? exp2f(-8.f * (h + 1) / a.heads) : 0.f;
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

// 16 bytes of a row starting at element `c` of `n`; elements at or beyond n are zero.
template <bool kAligned>
__device__ __forceinline__ void load_chunk(const __nv_bfloat16* p, int c, int n, float* f) {
  if (kAligned) {
    uint4 u = make_uint4(0, 0, 0, 0);
    if (c < n) u = *reinterpret_cast<const uint4*>(p + c);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 t = __bfloat1622float2(h[i]);
      f[2 * i] = t.x, f[2 * i + 1] = t.y;
    }
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = c + i < n ? __bfloat162float(p[c + i]) : 0.f;
  }
}
template <bool kAligned>
__device__ __forceinline__ void load_chunk(const float* p, int c, int n, float* f) {
  if (kAligned) {
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < n) u = *reinterpret_cast<const float4*>(p + c);
    f[0] = u.x, f[1] = u.y, f[2] = u.z, f[3] = u.w;
  } else {
#pragma unroll
    for (int i = 0; i < 4; ++i) f[i] = c + i < n ? p[c + i] : 0.f;
  }
}
// A lane's share of a head row: E elements in 16-byte chunks, chunk i at (lane8 + 8 i) * chunk size.
template <typename T, int E, bool kAligned>
__device__ __forceinline__ void load_share(const T* row, int lane8, int n, float (&f)[E]) {
  constexpr int VEC = 16 / sizeof(T);
#pragma unroll
  for (int i = 0; i < E / VEC; ++i) load_chunk<kAligned>(row, (lane8 + 8 * i) * VEC, n, f + i * VEC);
}

constexpr int kWdThreads = 128;

}  // namespace

// Eight lanes share a key; a warp covers four keys, the CTA sixteen.  GT query heads of one KV head.
template <typename T, int GT, int EK, int EV, bool kAligned>
__global__ void __launch_bounds__(kWdThreads) window_decode_kernel(WindowArgs a) {
  constexpr int VEC = 16 / sizeof(T);
  constexpr int U = EK <= 8 ? 4 : EK <= 16 ? (GT == 1 ? 4 : 2) : 1;  // keys per lane group in flight
  const int split = blockIdx.x, b = blockIdx.z;
  const int per_kv = a.heads / a.kv_heads, groups = per_kv / GT;
  const int kvh = blockIdx.y / groups, qh0 = kvh * per_kv + (blockIdx.y % groups) * GT;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, slot4 = lane >> 3, lane8 = lane & 7;
  const int pos = a.start[b];
  T* out = static_cast<T*>(a.out) + static_cast<int64_t>(b) * a.out_ld;
  if (pos < 0 || (a.live != nullptr && a.live[b] <= 0)) {  // row not in this step
    if (split == 0)
      for (int c = threadIdx.x; c < GT * a.vdim; c += kWdThreads) out[qh0 * a.vdim + c] = T(0.f);
    return;
  }
  const T* row = static_cast<const T*>(a.proj) + static_cast<int64_t>(b) * a.ld;
  T* k_ring = static_cast<T*>(a.k_ring) + static_cast<int64_t>(b) * a.slots * a.kv_heads * a.dim;
  T* v_ring = static_cast<T*>(a.v_ring) + static_cast<int64_t>(b) * a.slots * a.kv_heads * a.vdim;
  const T* k_new = row + a.k_off + kvh * a.dim;
  const T* v_new = row + a.v_off + kvh * a.vdim;
  if (split == 0 && blockIdx.y % groups == 0) {
    // The slot being written holds the key that has just left the window: nobody reads it.
    const int s = pos % a.slots;
    T* kd = k_ring + (static_cast<int64_t>(s) * a.kv_heads + kvh) * a.dim;
    T* vd = v_ring + (static_cast<int64_t>(s) * a.kv_heads + kvh) * a.vdim;
    for (int c = threadIdx.x; c < a.dim; c += kWdThreads) kd[c] = k_new[c];
    for (int c = threadIdx.x; c < a.vdim; c += kWdThreads) vd[c] = v_new[c];
  }
  const int lo = max(0, pos + 1 - min(a.window, a.slots));
  const int count = pos - lo + 1;
  const int per = (count + a.splits - 1) / a.splits;
  const int j_lo = lo + split * per, j_hi = min(pos + 1, j_lo + per);

  float q[GT][EK], acc[GT][EV], m[GT], l[GT], slope[GT];
  const float qs = query_scale(a, pos) * 1.4426950408889634f;
#pragma unroll
  for (int g = 0; g < GT; ++g) {
    load_share<T, EK, kAligned>(row + a.q_off + (qh0 + g) * a.dim, lane8, a.dim, q[g]);
#pragma unroll
    for (int i = 0; i < EK; ++i) q[g][i] *= qs;
#pragma unroll
    for (int i = 0; i < EV; ++i) acc[g][i] = 0.f;
    m[g] = -INFINITY, l[g] = 0.f;
    slope[g] = head_slope(a, qh0 + g) * 1.4426950408889634f;
  }
  for (int j0 = j_lo + warp * 4 + slot4; j0 - slot4 < j_hi; j0 += 16 * U) {
    float kf[U][EK], vf[U][EV];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int j = j0 + 16 * u;
      if (j < j_hi) {
        const int s = j % a.slots;
        const T* kp = j == pos ? k_new : k_ring + (static_cast<int64_t>(s) * a.kv_heads + kvh) * a.dim;
        const T* vp = j == pos ? v_new : v_ring + (static_cast<int64_t>(s) * a.kv_heads + kvh) * a.vdim;
        load_share<T, EK, kAligned>(kp, lane8, a.dim, kf[u]);
        load_share<T, EV, kAligned>(vp, lane8, a.vdim, vf[u]);
      } else {
#pragma unroll
        for (int i = 0; i < EK; ++i) kf[u][i] = 0.f;
#pragma unroll
        for (int i = 0; i < EV; ++i) vf[u][i] = 0.f;
      }
    }
#pragma unroll
    for (int g = 0; g < GT; ++g) {
      float s[U], mx = m[g];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int j = j0 + 16 * u;
        float d = 0.f;
#pragma unroll
        for (int i = 0; i < EK; ++i) d += q[g][i] * kf[u][i];
        d += __shfl_xor_sync(0xffffffffu, d, 1);
        d += __shfl_xor_sync(0xffffffffu, d, 2);
        d += __shfl_xor_sync(0xffffffffu, d, 4);
        s[u] = j < j_hi ? d - slope[g] * static_cast<float>(pos - j) : -INFINITY;
        mx = fmaxf(mx, s[u]);
      }
      const bool none = mx == -INFINITY;  // no key for this lane group yet
      const float corr = none ? 1.f : exp2f(m[g] - mx);
      l[g] *= corr;
#pragma unroll
      for (int i = 0; i < EV; ++i) acc[g][i] *= corr;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const float p = none ? 0.f : exp2f(s[u] - mx);
        l[g] += p;
#pragma unroll
        for (int i = 0; i < EV; ++i) acc[g][i] += p * vf[u][i];
      }
      m[g] = mx;
    }
  }

  // Four lane groups of a warp, then four warps.
  __shared__ float s_m[4][GT], s_l[4][GT], s_acc[4][GT][8 * EV];
  __shared__ int s_last;
#pragma unroll
  for (int g = 0; g < GT; ++g) {
#pragma unroll
    for (int off = 8; off <= 16; off <<= 1) {
      const float mo = __shfl_xor_sync(0xffffffffu, m[g], off), lo_ = __shfl_xor_sync(0xffffffffu, l[g], off);
      const float mn = fmaxf(m[g], mo);
      const float cs = mn == -INFINITY ? 1.f : exp2f(m[g] - mn), co = mn == -INFINITY ? 1.f : exp2f(mo - mn);
      l[g] = l[g] * cs + lo_ * co;
#pragma unroll
      for (int i = 0; i < EV; ++i)
        acc[g][i] = acc[g][i] * cs + __shfl_xor_sync(0xffffffffu, acc[g][i], off) * co;
      m[g] = mn;
    }
    if (slot4 == 0) {
#pragma unroll
      for (int i = 0; i < EV; ++i) s_acc[warp][g][(lane8 + 8 * (i / VEC)) * VEC + i % VEC] = acc[g][i];
      if (lane8 == 0) s_m[warp][g] = m[g], s_l[warp][g] = l[g];
    }
  }
  __syncthreads();
  const int pitch = a.vdim + 2;
#pragma unroll
  for (int g = 0; g < GT; ++g) {
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, s_m[w][g]);
    float c[4], ll = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      c[w] = mm == -INFINITY ? 0.f : exp2f(s_m[w][g] - mm);
      ll += s_l[w][g] * c[w];
    }
    float* part = a.splits == 1 ? nullptr
                                : a.part + ((static_cast<int64_t>(b) * a.heads + qh0 + g) * a.splits + split) * pitch;
    for (int d = threadIdx.x; d < a.vdim; d += kWdThreads) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) o += s_acc[w][g][d] * c[w];
      if (a.splits == 1) {
        o /= ll;
        const int col = (qh0 + g) * a.vdim + d;
        if (a.g_off >= 0) o *= sigmoid_f(to_f(row[a.g_off + col]));
        out[col] = T(o);
      } else {
        part[d] = o;
      }
    }
    if (a.splits > 1 && threadIdx.x == 0) part[a.vdim] = mm, part[a.vdim + 1] = ll;
  }
  if (a.splits == 1) return;
  // The last CTA of this (sequence, head group) merges the splits.
  __threadfence();
  __syncthreads();
  int* ticket = a.tickets + b * gridDim.y + blockIdx.y;
  if (threadIdx.x == 0) s_last = atomicAdd(ticket, 1) == a.splits - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  if (threadIdx.x == 0) *ticket = 0;
#pragma unroll 1
  for (int g = 0; g < GT; ++g) {
    const float* base = a.part + (static_cast<int64_t>(b) * a.heads + qh0 + g) * a.splits * pitch;
    float mm = -INFINITY;
    for (int s = 0; s < a.splits; ++s) mm = fmaxf(mm, __ldcg(base + s * pitch + a.vdim));
    float ll = 0.f;
    for (int s = 0; s < a.splits; ++s)
      ll += __ldcg(base + s * pitch + a.vdim + 1) * exp2f(__ldcg(base + s * pitch + a.vdim) - mm);
    for (int d = threadIdx.x; d < a.vdim; d += kWdThreads) {
      float o = 0.f;
      for (int s = 0; s < a.splits; ++s) o += __ldcg(base + s * pitch + d) * exp2f(__ldcg(base + s * pitch + a.vdim) - mm);
      o /= ll;
      const int col = (qh0 + g) * a.vdim + d;
      if (a.g_off >= 0) o *= sigmoid_f(to_f(row[a.g_off + col]));
      out[col] = T(o);
    }
  }
}

constexpr int kWaQ = 16, kWaK = 32, kWaThreads = 128;

// 16 queries of one head per CTA, keys in blocks of 32, everything fp32 in shared memory.
template <typename T>
__global__ void __launch_bounds__(kWaThreads) window_attn_kernel(WindowArgs a) {
  extern __shared__ float smem[];
  const int h = blockIdx.y, b = blockIdx.z, t0 = blockIdx.x * kWaQ;
  const int kvh = h / (a.heads / a.kv_heads);
  const int start = a.start != nullptr ? a.start[b] : 0;
  const int live = a.live != nullptr ? min(a.live[b], a.T) : a.T;
  const int kp = a.dim + 1;
  float* sq = smem;                      // [16][dim]
  float* sk = sq + kWaQ * a.dim;         // [32][dim + 1]
  float* sv = sk + kWaK * kp;            // [32][vdim]
  float* so = sv + kWaK * a.vdim;        // [16][vdim]
  float* ss = so + kWaQ * a.vdim;        // [16][33]
  float* sm = ss + kWaQ * (kWaK + 1);    // [16] running maximum
  float* sl = sm + kWaQ;                 // [16] running sum
  float* sc = sl + kWaQ;                 // [16] correction of this block
  T* out = static_cast<T*>(a.out);
  const int tid = threadIdx.x;
  if (t0 >= live || start < 0) {
    for (int i = tid; i < kWaQ * a.vdim; i += kWaThreads) {
      const int t = t0 + i / a.vdim;
      if (t < a.T) out[(static_cast<int64_t>(b) * a.T + t) * a.out_ld + h * a.vdim + i % a.vdim] = T(0.f);
    }
    return;
  }
  const T* proj = static_cast<const T*>(a.proj) + static_cast<int64_t>(b) * a.T * a.ld;
  const T* k_ring = static_cast<const T*>(a.k_ring) + static_cast<int64_t>(b) * a.slots * a.kv_heads * a.dim;
  const T* v_ring = static_cast<const T*>(a.v_ring) + static_cast<int64_t>(b) * a.slots * a.kv_heads * a.vdim;
  for (int i = tid; i < kWaQ * a.dim; i += kWaThreads) {
    const int r = i / a.dim, t = t0 + r;
    sq[i] = t < live ? to_f(proj[t * a.ld + a.q_off + h * a.dim + i % a.dim]) * query_scale(a, start + t) : 0.f;
  }
  for (int i = tid; i < kWaQ * a.vdim; i += kWaThreads) so[i] = 0.f;
  if (tid < kWaQ) sm[tid] = -INFINITY, sl[tid] = 0.f;
  const float slope = head_slope(a, h);
  const int first = start + t0, last = start + min(t0 + kWaQ, live) - 1;  // query positions of this CTA
  // Keys before `start` are in the ring, which holds the last `slots` of them.
  const int lo = max(max(0, first + 1 - a.window), start - a.slots);
  for (int j0 = lo; j0 <= last; j0 += kWaK) {
    const int n = min(kWaK, last - j0 + 1);
    __syncthreads();
    for (int i = tid; i < kWaK * a.dim; i += kWaThreads) {
      const int r = i / a.dim, c = i % a.dim, j = j0 + r;
      float x = 0.f;
      if (r < n)
        x = to_f(j < start ? k_ring[(static_cast<int64_t>(j % a.slots) * a.kv_heads + kvh) * a.dim + c]
                           : proj[(j - start) * a.ld + a.k_off + kvh * a.dim + c]);
      sk[r * kp + c] = x;
    }
    for (int i = tid; i < kWaK * a.vdim; i += kWaThreads) {
      const int r = i / a.vdim, c = i % a.vdim, j = j0 + r;
      float x = 0.f;
      if (r < n)
        x = to_f(j < start ? v_ring[(static_cast<int64_t>(j % a.slots) * a.kv_heads + kvh) * a.vdim + c]
                           : proj[(j - start) * a.ld + a.v_off + kvh * a.vdim + c]);
      sv[i] = x;
    }
    __syncthreads();
    const int col = tid & 31;
    for (int r = tid >> 5; r < kWaQ; r += kWaThreads / 32) {
      const int i = first + r, j = j0 + col;
      float s = -INFINITY;
      if (t0 + r < live && col < n && j <= i && i - j < a.window) {
        float d = 0.f;
        for (int c = 0; c < a.dim; ++c) d += sq[r * a.dim + c] * sk[col * kp + c];
        s = d - slope * static_cast<float>(i - j);
      }
      float mx = s;
      for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_old = sm[r], m_new = fmaxf(m_old, mx);
      const float p = s == -INFINITY ? 0.f : expf(s - m_new);
      float sum = p;
      for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      ss[r * (kWaK + 1) + col] = p;
      __syncwarp();
      if (col == 0) {
        const float c = m_old == -INFINITY ? 0.f : expf(m_old - m_new);
        sc[r] = c, sm[r] = m_new, sl[r] = sl[r] * c + sum;
      }
      __syncwarp();
    }
    __syncthreads();
    for (int i = tid; i < kWaQ * a.vdim; i += kWaThreads) {
      const int r = i / a.vdim, c = i % a.vdim;
      float o = so[i] * sc[r];
      for (int j = 0; j < n; ++j) o += ss[r * (kWaK + 1) + j] * sv[j * a.vdim + c];
      so[i] = o;
    }
  }
  __syncthreads();
  for (int i = tid; i < kWaQ * a.vdim; i += kWaThreads) {
    const int r = i / a.vdim, t = t0 + r;
    if (t >= a.T) continue;
    const int col = h * a.vdim + i % a.vdim;
    float o = 0.f;
    if (t < live) {
      o = so[i] / sl[r];
      if (a.g_off >= 0) o *= sigmoid_f(to_f(proj[t * a.ld + a.g_off + col]));
    }
    out[(static_cast<int64_t>(b) * a.T + t) * a.out_ld + col] = T(o);
  }
}

template <typename T>
__global__ void window_append_kernel(WindowArgs a) {
  const int b = blockIdx.y;
  const int start = a.start != nullptr ? a.start[b] : 0;
  const int live = a.live != nullptr ? min(a.live[b], a.T) : a.T;
  const int t = live - 1 - static_cast<int>(blockIdx.x);
  if (t < 0 || start < 0) return;
  const T* row = static_cast<const T*>(a.proj) + (static_cast<int64_t>(b) * a.T + t) * a.ld;
  const int64_t slot = static_cast<int64_t>(b) * a.slots + (start + t) % a.slots;
  T* kd = static_cast<T*>(a.k_ring) + slot * a.kv_heads * a.dim;
  T* vd = static_cast<T*>(a.v_ring) + slot * a.kv_heads * a.vdim;
  for (int c = threadIdx.x; c < a.kv_heads * a.dim; c += blockDim.x) kd[c] = row[a.k_off + c];
  for (int c = threadIdx.x; c < a.kv_heads * a.vdim; c += blockDim.x) vd[c] = row[a.v_off + c];
}

template <typename T>
__global__ void zero_columns_kernel(T* out, int64_t rows, int64_t ld, int first) {
  const int pad = static_cast<int>(ld) - first;
  const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i < rows * pad) out[(i / pad) * ld + first + i % pad] = T(0.f);
}

template <typename T>
static int zero_tail(const WindowArgs& a, cudaStream_t stream) {
  const int used = a.heads * a.vdim;
  if (a.out_ld == used) return 0;
  const int64_t rows = static_cast<int64_t>(a.B) * a.T, n = rows * (a.out_ld - used);
  zero_columns_kernel<T><<<static_cast<unsigned>((n + 255) / 256), 256, 0, stream>>>(static_cast<T*>(a.out), rows,
                                                                                     a.out_ld, used);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

static int query_heads_per_cta(int heads, int kv_heads) {
  const int per_kv = heads / kv_heads;
  return per_kv % 4 == 0 ? 4 : per_kv % 2 == 0 ? 2 : 1;
}

template <typename T, int GT, int EK, int EV>
static int launch_decode(const WindowArgs& a, bool aligned, cudaStream_t stream) {
  const dim3 grid(a.splits, a.heads / GT, a.B);
  if (aligned)
    window_decode_kernel<T, GT, EK, EV, true><<<grid, kWdThreads, 0, stream>>>(a);
  else
    window_decode_kernel<T, GT, EK, EV, false><<<grid, kWdThreads, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? zero_tail<T>(a, stream) : -4;
}

template <typename T, int GT>
static int dispatch_decode(const WindowArgs& a, bool aligned, cudaStream_t stream) {
  const int e = (a.dim > a.vdim ? a.dim : a.vdim);
  if (e <= 64) return launch_decode<T, GT, 8, 8>(a, aligned, stream);
  if (e <= 128) return launch_decode<T, GT, 16, 16>(a, aligned, stream);
  if (e <= 256) return launch_decode<T, (GT > 2 ? 2 : GT), 32, 32>(a, aligned, stream);
  return launch_decode<T, 1, 64, 64>(a, aligned, stream);
}

template <typename T>
static int window_decode(const WindowArgs& a, cudaStream_t stream) {
  constexpr int VEC = 16 / sizeof(T);
  auto ok = [](int64_t x) { return x % VEC == 0; };
  const bool aligned = ok(a.dim) && ok(a.vdim) && ok(a.ld) && ok(a.q_off) && ok(a.k_off) && ok(a.v_off);
  switch (query_heads_per_cta(a.heads, a.kv_heads)) {
    case 4: return dispatch_decode<T, 4>(a, aligned, stream);
    case 2: return dispatch_decode<T, 2>(a, aligned, stream);
    default: return dispatch_decode<T, 1>(a, aligned, stream);
  }
}

template <typename T>
static int window_attn(const WindowArgs& a, cudaStream_t stream) {
  const size_t smem = sizeof(float) * (kWaQ * a.dim + kWaK * (a.dim + 1) + kWaK * a.vdim + kWaQ * a.vdim +
                                       kWaQ * (kWaK + 1) + 3 * kWaQ);
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    if (smem > 220 * 1024 || cudaFuncSetAttribute(window_attn_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                  static_cast<int>(smem)) != cudaSuccess)
      return -3;
    configured = smem;
  }
  const dim3 grid((a.T + kWaQ - 1) / kWaQ, a.heads, a.B);
  window_attn_kernel<T><<<grid, kWaThreads, smem, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? zero_tail<T>(a, stream) : -4;
}

static bool bad(const WindowArgs& a) {
  return a.B <= 0 || a.T <= 0 || a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dim <= 0 ||
         a.vdim <= 0 || a.dim > 512 || a.vdim > 512 || a.slots <= 0 || a.window <= 0 || a.every <= 0 ||
         a.out_ld < static_cast<int64_t>(a.heads) * a.vdim || a.B > 65535 || a.heads > 65535;
}

}  // namespace axb

// CTAs of one KV split of the decode kernel (the caller sizes `splits` and `tickets` by it).
extern "C" int axb_window_decode_ctas(int B, int heads, int kv_heads, int dim, int vdim) {
  int gt = axb::query_heads_per_cta(heads, kv_heads);
  const int e = dim > vdim ? dim : vdim;
  if (e > 128 && gt > 2) gt = 2;
  if (e > 256) gt = 1;
  return B * (heads / gt);
}

// One new token per sequence (T == 1, `start` required).
extern "C" int axb_window_decode(const axb::WindowArgs* args, cudaStream_t stream) {
  const axb::WindowArgs& a = *args;
  if (axb::bad(a) || a.T != 1 || a.start == nullptr || a.splits < 1) return -10;
  if (a.splits > 1 && (a.part == nullptr || a.tickets == nullptr)) return -11;
  return a.act_bf16 ? axb::window_decode<__nv_bfloat16>(a, stream) : axb::window_decode<float>(a, stream);
}

// Attention of T new tokens per sequence over the ring and themselves; does not touch the ring.
extern "C" int axb_window_attn(const axb::WindowArgs* args, cudaStream_t stream) {
  const axb::WindowArgs& a = *args;
  if (axb::bad(a)) return -10;
  return a.act_bf16 ? axb::window_attn<__nv_bfloat16>(a, stream) : axb::window_attn<float>(a, stream);
}

// Stores the last `slots` live tokens into the ring.
extern "C" int axb_window_append(const axb::WindowArgs* args, cudaStream_t stream) {
  const axb::WindowArgs& a = *args;
  if (axb::bad(a)) return -10;
  const dim3 grid(a.T < a.slots ? a.T : a.slots, a.B);
  if (a.act_bf16)
    axb::window_append_kernel<__nv_bfloat16><<<grid, 128, 0, stream>>>(a);
  else
    axb::window_append_kernel<float><<<grid, 128, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
