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
  float* part;           // decode splits: [B, H, splits, vdim + 2 rounded up to 4]
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

// 16 bytes of a row starting at element `c` of `n`, raw; elements at or beyond n are zero.
template <typename T, bool kAligned>
__device__ __forceinline__ uint4 load_raw(const T* p, int c, int n) {
  uint4 u = make_uint4(0, 0, 0, 0);
  if (kAligned) {
    if (c < n) u = *reinterpret_cast<const uint4*>(p + c);
  } else {
    T* e = reinterpret_cast<T*>(&u);
#pragma unroll
    for (int i = 0; i < static_cast<int>(16 / sizeof(T)); ++i)
      if (c + i < n) e[i] = p[c + i];
  }
  return u;
}
template <typename T>
__device__ __forceinline__ void expand(const uint4& u, float* f);
template <>
__device__ __forceinline__ void expand<__nv_bfloat16>(const uint4& u, float* f) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 t = __bfloat1622float2(h[i]);
    f[2 * i] = t.x, f[2 * i + 1] = t.y;
  }
}
template <>
__device__ __forceinline__ void expand<float>(const uint4& u, float* f) {
  f[0] = __uint_as_float(u.x), f[1] = __uint_as_float(u.y), f[2] = __uint_as_float(u.z), f[3] = __uint_as_float(u.w);
}

constexpr int kWdThreads = 256, kWdWarps = kWdThreads / 32, kMaxSplits = 64;

}  // namespace

// LPK lanes share a key, NC 16-byte chunks of the head row each (chunk i of lane l at (l + LPK i) * 16
// bytes); a warp covers 32 / LPK keys per step and keeps U steps' loads in flight.  GT query heads of one KV
// head per CTA.
template <typename T, int GT, int LPK, int NC, int U, bool kAligned>
__global__ void __launch_bounds__(kWdThreads, 2) window_decode_kernel(WindowArgs a) {
  constexpr int VEC = 16 / sizeof(T);
  constexpr int E = NC * VEC;                // elements per lane
  constexpr int KPW = 32 / LPK;              // keys per warp and step
  constexpr int STEP = KPW * kWdWarps;
  const int split = blockIdx.x, b = blockIdx.z;
  const int per_kv = a.heads / a.kv_heads, groups = per_kv / GT;
  const int kvh = blockIdx.y / groups, qh0 = kvh * per_kv + (blockIdx.y % groups) * GT;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, slot = lane / LPK, lk = lane % LPK;
  const int pos = a.start[b];
  T* out = static_cast<T*>(a.out) + static_cast<int64_t>(b) * a.out_ld;
  if (pos < 0 || (a.live != nullptr && a.live[b] <= 0)) {  // row not in this step
    if (split == 0)
      for (int c = threadIdx.x; c < GT * a.vdim; c += kWdThreads) out[qh0 * a.vdim + c] = T(0.f);
    return;
  }
  const T* row = static_cast<const T*>(a.proj) + static_cast<int64_t>(b) * a.ld;
  T* k_ring = static_cast<T*>(a.k_ring) + (static_cast<int64_t>(b) * a.slots * a.kv_heads + kvh) * a.dim;
  T* v_ring = static_cast<T*>(a.v_ring) + (static_cast<int64_t>(b) * a.slots * a.kv_heads + kvh) * a.vdim;
  const int64_t k_pitch = static_cast<int64_t>(a.kv_heads) * a.dim, v_pitch = static_cast<int64_t>(a.kv_heads) * a.vdim;
  const T* k_new = row + a.k_off + kvh * a.dim;
  const T* v_new = row + a.v_off + kvh * a.vdim;
  const int lo = max(0, pos + 1 - min(a.window, a.slots));
  const int count = pos - lo + 1;
  const int per = (count + a.splits - 1) / a.splits;
  const int j_lo = lo + split * per, j_hi = min(pos + 1, j_lo + per);

  float q[GT][E], acc[GT][E], m[GT], l[GT], slope[GT];
  const float qs = query_scale(a, pos) * 1.4426950408889634f;
#pragma unroll
  for (int g = 0; g < GT; ++g) {
#pragma unroll
    for (int i = 0; i < NC; ++i)
      expand<T>(load_raw<T, kAligned>(row + a.q_off + (qh0 + g) * a.dim, (lk + LPK * i) * VEC, a.dim), q[g] + i * VEC);
#pragma unroll
    for (int i = 0; i < E; ++i) q[g][i] *= qs, acc[g][i] = 0.f;
    m[g] = -INFINITY, l[g] = 0.f;
    slope[g] = head_slope(a, qh0 + g) * 1.4426950408889634f;
  }
  // Ring slot of a key, kept by addition: a step moves every lane group by STEP keys.
  int j = j_lo + warp * KPW + slot;
  int at = j % a.slots;
  const int step_slots = STEP % a.slots;
  for (; j - slot < j_hi;) {
    uint4 kr[U][NC], vr[U][NC];
    bool ok[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int ju = j + STEP * u;
      ok[u] = ju < j_hi;
      const T* kp = ju == pos ? k_new : k_ring + at * k_pitch;
      const T* vp = ju == pos ? v_new : v_ring + at * v_pitch;
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        kr[u][i] = vr[u][i] = make_uint4(0, 0, 0, 0);
        if (ok[u]) {
          kr[u][i] = load_raw<T, kAligned>(kp, (lk + LPK * i) * VEC, a.dim);
          vr[u][i] = load_raw<T, kAligned>(vp, (lk + LPK * i) * VEC, a.vdim);
        }
      }
      at += step_slots;
      if (at >= a.slots) at -= a.slots;
    }
    float s[GT][U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float kf[E];
#pragma unroll
      for (int i = 0; i < NC; ++i) expand<T>(kr[u][i], kf + i * VEC);
#pragma unroll
      for (int g = 0; g < GT; ++g) {
        float d = 0.f;
#pragma unroll
        for (int i = 0; i < E; ++i) d += q[g][i] * kf[i];
        s[g][u] = d;
      }
    }
#pragma unroll
    for (int off = 1; off < LPK; off <<= 1)
#pragma unroll
      for (int g = 0; g < GT; ++g)
#pragma unroll
        for (int u = 0; u < U; ++u) s[g][u] += __shfl_xor_sync(0xffffffffu, s[g][u], off);
#pragma unroll
    for (int g = 0; g < GT; ++g) {
      float mx = m[g];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        s[g][u] = ok[u] ? s[g][u] - slope[g] * static_cast<float>(pos - j - STEP * u) : -INFINITY;
        mx = fmaxf(mx, s[g][u]);
      }
      const bool none = mx == -INFINITY;  // no key for this lane group yet
      const float corr = none ? 1.f : exp2f(m[g] - mx);
      l[g] *= corr;
#pragma unroll
      for (int i = 0; i < E; ++i) acc[g][i] *= corr;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        s[g][u] = none ? 0.f : exp2f(s[g][u] - mx);
        l[g] += s[g][u];
      }
      m[g] = mx;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float vf[E];
#pragma unroll
      for (int i = 0; i < NC; ++i) expand<T>(vr[u][i], vf + i * VEC);
#pragma unroll
      for (int g = 0; g < GT; ++g)
#pragma unroll
        for (int i = 0; i < E; ++i) acc[g][i] += s[g][u] * vf[i];
    }
    j += STEP * U;
  }
  if (split == 0 && blockIdx.y % groups == 0) {
    // The slot being written holds the key that has just left the window: nobody reads it.
    const int64_t s = pos % a.slots;
    for (int c = threadIdx.x; c < a.dim; c += kWdThreads) k_ring[s * k_pitch + c] = k_new[c];
    for (int c = threadIdx.x; c < a.vdim; c += kWdThreads) v_ring[s * v_pitch + c] = v_new[c];
  }

  // Lane groups of a warp, then the warps.
  __shared__ float s_m[kWdWarps][GT], s_l[kWdWarps][GT], s_acc[kWdWarps][GT][LPK * E];
  __shared__ float s_c[GT][kWdWarps];
  __shared__ int s_last;
#pragma unroll
  for (int g = 0; g < GT; ++g) {
#pragma unroll
    for (int off = LPK; off < 32; off <<= 1) {
      const float mo = __shfl_xor_sync(0xffffffffu, m[g], off), lo_ = __shfl_xor_sync(0xffffffffu, l[g], off);
      const float mn = fmaxf(m[g], mo);
      const float cs = mn == -INFINITY ? 1.f : exp2f(m[g] - mn), co = mn == -INFINITY ? 1.f : exp2f(mo - mn);
      l[g] = l[g] * cs + lo_ * co;
#pragma unroll
      for (int i = 0; i < E; ++i)
        acc[g][i] = acc[g][i] * cs + __shfl_xor_sync(0xffffffffu, acc[g][i], off) * co;
      m[g] = mn;
    }
    if (slot == 0) {
#pragma unroll
      for (int i = 0; i < E; ++i) s_acc[warp][g][(lk + LPK * (i / VEC)) * VEC + i % VEC] = acc[g][i];
      if (lk == 0) s_m[warp][g] = m[g], s_l[warp][g] = l[g];
    }
  }
  __syncthreads();
  const int pitch = (a.vdim + 5) & ~3;  // outputs, then maximum and sum
  float* part = a.part + (static_cast<int64_t>(b) * a.heads + qh0) * a.splits * pitch;  // [GT][splits][pitch]
  if (threadIdx.x < GT) {
    const int g = threadIdx.x;
    float mm = -INFINITY, ll = 0.f;
    for (int w = 0; w < kWdWarps; ++w) mm = fmaxf(mm, s_m[w][g]);
    for (int w = 0; w < kWdWarps; ++w) {
      const float c = mm == -INFINITY ? 0.f : exp2f(s_m[w][g] - mm);
      ll += s_l[w][g] * c;
      s_c[g][w] = c;
    }
    if (a.splits == 1) {
      for (int w = 0; w < kWdWarps; ++w) s_c[g][w] /= ll;
    } else {
      float* mine = part + (g * a.splits + split) * pitch + a.vdim;
      mine[0] = mm, mine[1] = ll;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < GT * a.vdim; i += kWdThreads) {
    const int g = i / a.vdim, d = i % a.vdim;
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < kWdWarps; ++w) o += s_acc[w][g][d] * s_c[g][w];
    if (a.splits == 1) {
      const int col = qh0 * a.vdim + i;
      if (a.g_off >= 0) o *= sigmoid_f(to_f(row[a.g_off + col]));
      out[col] = T(o);
    } else {
      part[(g * a.splits + split) * pitch + d] = o;
    }
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
  // Weight of every split: one warp per head.
  __shared__ float s_w[GT][kMaxSplits];
  if (warp < GT) {
    const int g = warp;
    float mv[kMaxSplits / 32], lv[kMaxSplits / 32], mm = -INFINITY, ll = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxSplits / 32; ++i) {
      const int s = lane + 32 * i;
      const float* p = part + (g * a.splits + s) * pitch + a.vdim;
      mv[i] = s < a.splits ? __ldcg(p) : -INFINITY;
      lv[i] = s < a.splits ? __ldcg(p + 1) : 0.f;
      mm = fmaxf(mm, mv[i]);
    }
    for (int off = 16; off > 0; off >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffffu, mm, off));
#pragma unroll
    for (int i = 0; i < kMaxSplits / 32; ++i) mv[i] = exp2f(mv[i] - mm), ll += lv[i] * mv[i];
    for (int off = 16; off > 0; off >>= 1) ll += __shfl_xor_sync(0xffffffffu, ll, off);
#pragma unroll
    for (int i = 0; i < kMaxSplits / 32; ++i) s_w[g][lane + 32 * i] = mv[i] / ll;
  }
  __syncthreads();
  auto finish = [&](int col, float o) {
    if (a.g_off >= 0) o *= sigmoid_f(to_f(row[a.g_off + col]));
    out[col] = T(o);
  };
  if (a.vdim % 4 == 0) {
    for (int i = threadIdx.x; i < GT * (a.vdim / 4); i += kWdThreads) {
      const int g = i / (a.vdim / 4), d = (i % (a.vdim / 4)) * 4;
      const float* p = part + g * a.splits * pitch + d;
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
      for (int s = 0; s < a.splits; ++s) {
        const float4 x = __ldcg(reinterpret_cast<const float4*>(p + s * pitch));
        const float w = s_w[g][s];
        o.x += x.x * w, o.y += x.y * w, o.z += x.z * w, o.w += x.w * w;
      }
      const int col = (qh0 + g) * a.vdim + d;
      finish(col, o.x), finish(col + 1, o.y), finish(col + 2, o.z), finish(col + 3, o.w);
    }
  } else {
    for (int i = threadIdx.x; i < GT * a.vdim; i += kWdThreads) {
      const int g = i / a.vdim;
      const float* p = part + g * a.splits * pitch + i % a.vdim;
      float o = 0.f;
      for (int s = 0; s < a.splits; ++s) o += __ldcg(p + s * pitch) * s_w[g][s];
      finish(qh0 * a.vdim + i, o);
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

// V: 16-byte vectors (row sizes, pitches and offsets permitting) or single elements.
template <typename V, typename T>
__global__ void __launch_bounds__(128) window_append_kernel(WindowArgs a) {
  constexpr int N = sizeof(V) / sizeof(T);
  const int b = blockIdx.y;
  const int start = a.start != nullptr ? a.start[b] : 0;
  const int live = a.live != nullptr ? min(a.live[b], a.T) : a.T;
  const int kc = a.kv_heads * a.dim / N, vc = a.kv_heads * a.vdim / N;
  for (int back = blockIdx.x; back < a.slots; back += gridDim.x) {
    const int t = live - 1 - back;
    if (t < 0 || start < 0) return;
    const T* row = static_cast<const T*>(a.proj) + (static_cast<int64_t>(b) * a.T + t) * a.ld;
    const int64_t slot = static_cast<int64_t>(b) * a.slots + (start + t) % a.slots;
    const V* ks = reinterpret_cast<const V*>(row + a.k_off);
    const V* vs = reinterpret_cast<const V*>(row + a.v_off);
    V* kd = reinterpret_cast<V*>(static_cast<T*>(a.k_ring)) + slot * kc;
    V* vd = reinterpret_cast<V*>(static_cast<T*>(a.v_ring)) + slot * vc;
    for (int c = threadIdx.x; c < kc + vc; c += blockDim.x) {
      if (c < kc)
        kd[c] = ks[c];
      else
        vd[c - kc] = vs[c - kc];
    }
  }
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

template <typename T, int GT, int LPK, int NC, int U>
static int launch_decode(const WindowArgs& a, bool aligned, cudaStream_t stream) {
  const dim3 grid(a.splits, a.heads / GT, a.B);
  if (aligned)
    window_decode_kernel<T, GT, LPK, NC, U, true><<<grid, kWdThreads, 0, stream>>>(a);
  else
    window_decode_kernel<T, GT, LPK, NC, U, false><<<grid, kWdThreads, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? zero_tail<T>(a, stream) : -4;
}

// Eight bf16 (or two times four fp32) elements per lane; 512-element heads take twice that.
template <typename T, int GT>
static int dispatch_decode(const WindowArgs& a, bool aligned, cudaStream_t stream) {
  constexpr int N = sizeof(T) / 2, U = (GT == 4 ? 2 : 4) / N;
  const int e = a.dim > a.vdim ? a.dim : a.vdim;
  if (e <= 64) return launch_decode<T, GT, 8, N, U>(a, aligned, stream);
  if (e <= 128) return launch_decode<T, GT, 16, N, U>(a, aligned, stream);
  if (e <= 256) return launch_decode<T, GT, 32, N, U>(a, aligned, stream);
  return launch_decode<T, (GT > 2 ? 2 : GT), 32, 2 * N, 1>(a, aligned, stream);
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

template <typename T>
static int window_append(const WindowArgs& a, cudaStream_t stream) {
  constexpr int VEC = 16 / sizeof(T);
  const int tokens = a.T < a.slots ? a.T : a.slots;
  const dim3 grid(tokens < 1024 ? tokens : 1024, a.B);
  auto ok = [](int64_t x) { return x % VEC == 0; };
  if (ok(a.ld) && ok(a.k_off) && ok(a.v_off) && ok(a.kv_heads * a.dim) && ok(a.kv_heads * a.vdim))
    window_append_kernel<uint4, T><<<grid, 128, 0, stream>>>(a);
  else
    window_append_kernel<T, T><<<grid, 128, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
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
  if ((dim > vdim ? dim : vdim) > 256 && gt > 2) gt = 2;
  return B * (heads / gt);
}

// One new token per sequence (T == 1, `start` required).
extern "C" int axb_window_decode(const axb::WindowArgs* args, cudaStream_t stream) {
  const axb::WindowArgs& a = *args;
  if (axb::bad(a) || a.T != 1 || a.start == nullptr || a.splits < 1 || a.splits > axb::kMaxSplits) return -10;
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
  return a.act_bf16 ? axb::window_append<__nv_bfloat16>(a, stream) : axb::window_append<float>(a, stream);
}
