// Latent attention: one cached row [latent | rotated key part] per token serves the keys and values of all
// heads.
//
// Cache rows are [row_w] = latent (rank columns, padded to rot_off) then the rotated part (padded); padding is
// zero.  With queries folded into the latent space (q_lat = W_uk^T q per head) attention is
//   score = q_row . cache_row * scale,  out_lat = softmax(score) . latents        over j <= position
// i.e. multi-query attention with a key size of row_w and a value size of rank.
//
// `start[b]` tokens are cached already (null: zero; < 0: row not in this step), `live[b]` of the T new ones are
// valid (null: T).
//
//   latent_prep_kernel    norm of the latent, rotation of the key part, cache row; rotation of the queries
//                         (in place, or into the rows that latent attention reads); latent_prep_vec_kernel is
//                         its form for aligned bf16 prompts.
//   latent_decode_kernel  bf16: 16 or 32 heads of one query token per CTA on the tensor cores, the cached rows
//                         streamed once through shared memory; long caches are split over CTAs and
//                         latent_merge_kernel joins the parts.
//   latent_attn_kernel    any sizes, fp32 or bf16, one CTA per (token, head).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "mma_sync.cuh"

namespace axb {

struct LatentArgs {
  const void* proj;      // queries are rotated in place without qbuf
  const float* norm_w;   // [rank]
  const double* freq;    // [rot_dims / 2]
  void* cache;           // [B, slots, cache_ld]
  void* lat;             // [B * T, lat_ld] normed latents of the new tokens, or null
  void* qbuf;            // [B * T, heads, row_w], or null
  void* out;             // [B * T, heads, out_ld]
  float* part;           // [B * T, heads, splits, rot_off] un-normalised sums
  float* part_ml;        // [B * T, heads, splits, 2] their score maximum (log2) and weight
  const int* start;
  const int* live;
  int64_t ld, cache_ld, lat_ld, out_ld;
  int B, T, heads, dim, rot_dim, rot_dims, rank, rot_off, row_w, slots;
  int q_off, c_off, r_off, splits, act_bf16;
  float scale, eps;
};

namespace {

__device__ __forceinline__ float lf(float x) { return x; }
__device__ __forceinline__ float lf(__nv_bfloat16 x) { return __bfloat162float(x); }
constexpr float kLog2E = 1.4426950408889634f;

// Position of token t of sequence b, -1 when it takes no part in the step.
__device__ __forceinline__ int token_position(const LatentArgs& a, int b, int t) {
  const int start = a.start != nullptr ? a.start[b] : 0;
  const int live = a.live != nullptr ? a.live[b] : a.T;
  return start < 0 || t >= live || start + t >= a.slots ? -1 : start + t;
}

constexpr int kLpThreads = 128;

}  // namespace

// blockIdx.z = 0: the latent and the key part; z > 0: queries of `heads_per` heads.
template <typename T>
__global__ void __launch_bounds__(kLpThreads) latent_prep_kernel(LatentArgs a, int heads_per) {
  extern __shared__ float2 s_turn[];  // (cos, sin) per pair
  __shared__ float red[kLpThreads / 32];
  const int t = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int64_t row = static_cast<int64_t>(b) * a.T + t;
  T* src = static_cast<T*>(const_cast<void*>(a.proj)) + row * a.ld;
  const int pos = token_position(a, b, t);
  const int half = a.rot_dims / 2;
  for (int i = tid; i < half; i += kLpThreads) {
    // The angle is reduced to one turn in double precision.
    const double turn = 6.283185307179586476925286766559;
    double angle = max(pos, 0) * a.freq[i];
    angle -= turn * rint(angle * (1.0 / turn));
    float s, c;
    sincosf(static_cast<float>(angle), &s, &c);
    s_turn[i] = make_float2(c, s);
  }
  // Element i of a rotated part, from its unrotated values.
  auto rotated = [&](const T* x, int i) {
    if (i >= a.rot_dims) return lf(x[i]);
    const float2 cs = s_turn[i >> 1];
    const float u = lf(x[i & ~1]), v = lf(x[i | 1]);
    return i & 1 ? v * cs.x + u * cs.y : u * cs.x - v * cs.y;
  };
  const int pad = a.row_w - a.rot_off;
  if (blockIdx.z == 0) {
    float sq = 0.f;
    for (int c = tid; c < a.rank; c += kLpThreads) {
      const float x = lf(src[a.c_off + c]);
      sq += x * x;
    }
    for (int off = 16; off > 0; off >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, off);
    if ((tid & 31) == 0) red[tid >> 5] = sq;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < kLpThreads / 32; ++w) total += red[w];
    const float inv = 1.f / sqrtf(total / a.rank + a.eps);
    T* dst = pos >= 0 ? static_cast<T*>(a.cache) + (static_cast<int64_t>(b) * a.slots + pos) * a.cache_ld : nullptr;
    T* lat = a.lat != nullptr ? static_cast<T*>(a.lat) + row * a.lat_ld : nullptr;
    for (int c = tid; c < a.rot_off; c += kLpThreads) {
      const T y = c < a.rank ? T(lf(src[a.c_off + c]) * inv * a.norm_w[c]) : T(0.f);
      if (dst != nullptr) dst[c] = y;
      if (lat != nullptr) lat[c] = y;
    }
    if (dst != nullptr)
      for (int i = tid; i < pad; i += kLpThreads) dst[a.rot_off + i] = i < a.rot_dim ? T(rotated(src + a.r_off, i)) : T(0.f);
    return;
  }
  __syncthreads();
  const int head_w = a.dim + a.rot_dim;
  const int h0 = (blockIdx.z - 1) * heads_per, heads = min(heads_per, a.heads - h0);
  src += a.q_off + h0 * head_w + a.dim;
  if (a.qbuf != nullptr) {
    T* q = static_cast<T*>(a.qbuf) + (row * a.heads + h0) * a.row_w + a.rot_off;
#pragma unroll 4
    for (int i = tid; i < heads * pad; i += kLpThreads) {
      const int h = i / pad, c = i % pad;
      q[h * a.row_w + c] = c < a.rot_dim ? T(rotated(src + h * head_w, c)) : T(0.f);
    }
  } else {
#pragma unroll 4
    for (int i = tid; i < heads * half; i += kLpThreads) {
      T* x = src + (i / half) * head_w + (i % half) * 2;
      const float2 cs = s_turn[i % half];
      const float u = lf(x[0]), v = lf(x[1]);
      x[0] = T(u * cs.x - v * cs.y);
      x[1] = T(v * cs.x + u * cs.y);
    }
  }
}

// Prompts with 16-byte aligned parts: four tokens per CTA, one warp each for the latent and one for the queries,
// which are rotated in place.
constexpr int kLvTokens = 4;

__global__ void __launch_bounds__(64 * kLvTokens) latent_prep_vec_kernel(LatentArgs a) {
  using bf16 = __nv_bfloat16;
  extern __shared__ float2 s_turn[];  // [4][rot_dims / 2] (cos, sin)
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, half = a.rot_dims / 2;
  const int64_t tokens = static_cast<int64_t>(a.B) * a.T, first = static_cast<int64_t>(blockIdx.x) * kLvTokens;
  for (int i = tid; i < kLvTokens * half; i += 64 * kLvTokens) {
    const int64_t row = min(first + i / half, tokens - 1);
    const int pos = token_position(a, static_cast<int>(row / a.T), static_cast<int>(row % a.T));
    const double turn = 6.283185307179586476925286766559;
    double angle = max(pos, 0) * a.freq[i % half];
    angle -= turn * rint(angle * (1.0 / turn));
    float s, c;
    sincosf(static_cast<float>(angle), &s, &c);
    s_turn[i] = make_float2(c, s);
  }
  const int64_t row = first + warp % kLvTokens;
  const float2* cs = s_turn + (warp % kLvTokens) * half;
  const bool valid = row < tokens;
  bf16* src = static_cast<bf16*>(const_cast<void*>(a.proj)) + (valid ? row : 0) * a.ld;
  // Eight consecutive elements from element c on of a rotated part.
  auto turn8 = [&](const uint4& u, int c) {
    const uint32_t in[4] = {u.x, u.y, u.z, u.w};
    uint32_t o[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 x = unpack2(in[i]);
      const float2 t = c + 2 * i < a.rot_dims ? cs[(c >> 1) + i] : make_float2(1.f, 0.f);
      o[i] = pack2(x.x * t.x - x.y * t.y, x.y * t.x + x.x * t.y);
    }
    return make_uint4(o[0], o[1], o[2], o[3]);
  };
  if (warp >= kLvTokens) {
    const int head_w = a.dim + a.rot_dim, per = a.rot_dim / 8, items = a.heads * per;
    bf16* q = src + a.q_off + a.dim;
    __syncthreads();
    if (!valid) return;
#pragma unroll 4
    for (int i = lane; i < items; i += 32) {
      const int c = i % per * 8;
      uint4* x = reinterpret_cast<uint4*>(q + static_cast<int64_t>(i / per) * head_w + c);
      *x = turn8(*x, c);
    }
    return;
  }
  const int b = static_cast<int>((valid ? row : 0) / a.T), t = static_cast<int>((valid ? row : 0) % a.T);
  const int pos = token_position(a, b, t);
  float sq = 0.f;
  for (int c = lane * 8; c < a.rank; c += 256) {
    const uint4 u = *reinterpret_cast<const uint4*>(src + a.c_off + c);
    const uint32_t in[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 x = unpack2(in[i]);
      sq += x.x * x.x + x.y * x.y;
    }
  }
  for (int off = 16; off > 0; off >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, off);
  const float inv = 1.f / sqrtf(sq / a.rank + a.eps);
  __syncthreads();
  if (!valid) return;
  bf16* dst = pos >= 0 ? static_cast<bf16*>(a.cache) + (static_cast<int64_t>(b) * a.slots + pos) * a.cache_ld : nullptr;
  bf16* lat = static_cast<bf16*>(a.lat) + row * a.lat_ld;
  for (int c = lane * 8; c < a.rank; c += 256) {
    const uint4 u = *reinterpret_cast<const uint4*>(src + a.c_off + c);
    const uint32_t in[4] = {u.x, u.y, u.z, u.w};
    const float4 w0 = *reinterpret_cast<const float4*>(a.norm_w + c), w1 = *reinterpret_cast<const float4*>(a.norm_w + c + 4);
    const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
    uint32_t o[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 x = unpack2(in[i]);
      o[i] = pack2(x.x * inv * w[2 * i], x.y * inv * w[2 * i + 1]);
    }
    const uint4 y = make_uint4(o[0], o[1], o[2], o[3]);
    if (dst != nullptr) *reinterpret_cast<uint4*>(dst + c) = y;
    *reinterpret_cast<uint4*>(lat + c) = y;
  }
  if (dst != nullptr)
    for (int c = lane * 8; c < a.rot_dim; c += 256)
      *reinterpret_cast<uint4*>(dst + a.rot_off + c) = turn8(*reinterpret_cast<const uint4*>(src + a.r_off + c), c);
}

constexpr int kLaThreads = 256, kLaKeys = 64, kLaCols = 8;

template <typename T>
__global__ void __launch_bounds__(kLaThreads) latent_attn_kernel(LatentArgs a) {
  extern __shared__ float s_q[];  // [row_w], times scale * log2(e)
  __shared__ float s_p[kLaKeys];
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int64_t row = blockIdx.x;
  const int b = static_cast<int>(row / a.T), t = static_cast<int>(row % a.T);
  T* out = static_cast<T*>(a.out) + (row * a.heads + h) * a.out_ld;
  const int pos = token_position(a, b, t);
  if (pos < 0) {
    for (int c = tid; c < a.rot_off; c += kLaThreads) out[c] = T(0.f);
    return;
  }
  const T* q = static_cast<const T*>(a.qbuf) + (row * a.heads + h) * a.row_w;
  for (int c = tid; c < a.row_w; c += kLaThreads) s_q[c] = lf(q[c]) * a.scale * kLog2E;
  const T* keys = static_cast<const T*>(a.cache) + static_cast<int64_t>(b) * a.slots * a.cache_ld;
  float acc[kLaCols], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int i = 0; i < kLaCols; ++i) acc[i] = 0.f;
  for (int j0 = 0; j0 <= pos; j0 += kLaKeys) {
    const int n = min(kLaKeys, pos + 1 - j0);
    __syncthreads();
    for (int j = warp; j < kLaKeys; j += kLaThreads / 32) {
      float s = 0.f;
      if (j < n) {
        const T* k = keys + static_cast<int64_t>(j0 + j) * a.cache_ld;
        for (int c = lane; c < a.row_w; c += 32) s += s_q[c] * lf(k[c]);
      }
      for (int off = 16; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
      if (lane == 0) s_p[j] = j < n ? s : -INFINITY;
    }
    __syncthreads();
    float mx = m;
    for (int j = 0; j < n; ++j) mx = fmaxf(mx, s_p[j]);
    const float corr = exp2f(m - mx);  // 0 for the first block
    l *= corr;
#pragma unroll
    for (int i = 0; i < kLaCols; ++i) acc[i] *= corr;
    m = mx;
    for (int j = 0; j < n; ++j) {
      const float p = exp2f(s_p[j] - mx);
      l += p;
      const T* v = keys + static_cast<int64_t>(j0 + j) * a.cache_ld;
#pragma unroll
      for (int i = 0; i < kLaCols; ++i) {
        const int c = tid + i * kLaThreads;
        if (c < a.rot_off) acc[i] += p * lf(v[c]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < kLaCols; ++i) {
    const int c = tid + i * kLaThreads;
    if (c < a.rot_off) out[c] = T(acc[i] / l);
  }
}

// ------------------------------------------------------------------------------------------
// Tensor-core form for a decoding step.
// ------------------------------------------------------------------------------------------
namespace {

constexpr int kLdThreads = 256, kLdWarps = 8, kLdKeys = 64, kLdMaxPairs = 4, kLdMaxSplits = 64;

__host__ __device__ constexpr int ld_width(int row_w) { return (row_w + 31) / 32 * 32; }

struct LdSmem {
  int q, k, stage, s, p, m, l, alpha, total;
};
__host__ __device__ inline LdSmem ld_smem(int row_w, int heads) {
  LdSmem x;
  const int pitch = (ld_width(row_w) + 8) * 2;
  x.q = 0;
  x.k = x.q + heads * pitch;
  x.stage = kLdKeys * pitch;
  x.s = x.k + 2 * x.stage;                     // float [heads][68]
  x.p = x.s + heads * (kLdKeys + 4) * 4;       // bf16 [heads][72]
  x.m = x.p + heads * (kLdKeys + 8) * 2;
  x.l = x.m + heads * 4;
  x.alpha = x.l + heads * 4;
  x.total = x.alpha + heads * 4;
  return x;
}

}  // namespace

// MT tiles of 16 heads per CTA.
template <int MT>
__global__ void __launch_bounds__(kLdThreads, 1) latent_decode_kernel(LatentArgs a) {
  using bf16 = __nv_bfloat16;
  constexpr int HB = MT * 16;
  extern __shared__ __align__(16) uint8_t ld_mem[];
  const LdSmem L = ld_smem(a.row_w, HB);
  const int WP = ld_width(a.row_w), pitch = WP + 8;
  bf16* sQ = reinterpret_cast<bf16*>(ld_mem + L.q);
  float* sS = reinterpret_cast<float*>(ld_mem + L.s);
  bf16* sP = reinterpret_cast<bf16*>(ld_mem + L.p);
  float* s_m = reinterpret_cast<float*>(ld_mem + L.m);
  float* s_l = reinterpret_cast<float*>(ld_mem + L.l);
  float* s_alpha = reinterpret_cast<float*>(ld_mem + L.alpha);
  constexpr int kSP = kLdKeys + 4, kPP = kLdKeys + 8;
  const int split = blockIdx.y, h0 = blockIdx.z * HB;
  const int64_t row = blockIdx.x;
  const int b = static_cast<int>(row / a.T), t = static_cast<int>(row % a.T);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lc = (lane & 3) * 2;
  const int nh = min(HB, a.heads - h0);
  bf16* out = static_cast<bf16*>(a.out) + (row * a.heads + h0) * a.out_ld;
  const int pos = token_position(a, b, t);
  if (pos < 0) {
    if (split == 0)
      for (int i = tid; i < nh * a.rot_off; i += kLdThreads)
        out[(i / a.rot_off) * a.out_ld + i % a.rot_off] = __float2bfloat16(0.f);
    return;
  }
  // Whole tiles of keys, shared out evenly over the splits.
  const int count = pos + 1, tiles = (count + kLdKeys - 1) / kLdKeys;
  const int j_lo = static_cast<int>(static_cast<int64_t>(split) * tiles / a.splits) * kLdKeys;
  const int j_hi = min(count, static_cast<int>(static_cast<int64_t>(split + 1) * tiles / a.splits) * kLdKeys);
  const bf16* keys = static_cast<const bf16*>(a.cache) + static_cast<int64_t>(b) * a.slots * a.cache_ld;
  const int chunks = WP / 8, valid = a.row_w / 8;  // 16-byte pieces of a row

  // A warp takes every eighth row, its lanes the pieces of the row.
  auto load_keys = [&](int j0, int stage) {
    bf16* dst = reinterpret_cast<bf16*>(ld_mem + L.k + stage * L.stage) + warp * pitch;
    const bf16* src = keys + static_cast<int64_t>(j0 + warp) * a.cache_ld;
#pragma unroll
    for (int r = 0; r < kLdKeys / kLdWarps; ++r) {
      const bool in = j0 + warp + r * kLdWarps < j_hi;
      for (int c = lane; c < chunks; c += 32) {
        if (in && c < valid)
          cp16(dst + c * 8, src + c * 8);
        else
          *reinterpret_cast<uint4*>(dst + c * 8) = make_uint4(0, 0, 0, 0);
      }
      dst += kLdWarps * pitch;
      src += kLdWarps * a.cache_ld;
    }
  };
  const bf16* q = static_cast<const bf16*>(a.qbuf) + (row * a.heads + h0) * a.row_w;
  for (int i = tid; i < HB * chunks; i += kLdThreads) {
    const int r = i / chunks, c = i % chunks;
    if (c < valid && r < nh)
      cp16(sQ + r * pitch + c * 8, q + static_cast<int64_t>(r) * a.row_w + c * 8);
    else
      *reinterpret_cast<uint4*>(sQ + r * pitch + c * 8) = make_uint4(0, 0, 0, 0);
  }
  load_keys(j_lo, 0);
  cp_commit();
  if (tid < HB) s_m[tid] = -INFINITY, s_l[tid] = 0.f;

  const int n_pairs = (a.rank + 15) / 16;  // 16-column tiles of the values, warp, warp + 8, ...
  float acc[MT][kLdMaxPairs][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < kLdMaxPairs; ++i)
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[m][i][u][e] = 0.f;
  const float sc = a.scale * kLog2E;

  for (int j0 = j_lo, it = 0; j0 < j_hi; j0 += kLdKeys, ++it) {
    const int stage = it & 1;
    if (j0 + kLdKeys < j_hi) load_keys(j0 + kLdKeys, stage ^ 1);
    cp_commit();
    cp_wait_group<1>();
    __syncthreads();
    const bf16* sK = reinterpret_cast<const bf16*>(ld_mem + L.k + stage * L.stage);
    {  // scores of keys [8 warp, + 8)
      float c0[MT][4], c1[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) c0[m][e] = c1[m][e] = 0.f;
      const bf16* kp = sK + (warp * 8 + (lane & 7)) * pitch + (lane >> 3) * 8;
      const bf16* qp = sQ + (lane & 15) * pitch + (lane >> 4) * 8;
#pragma unroll 4
      for (int k = 0; k < WP; k += 32) {
        uint32_t bk[4];
        ldsm4(bk, kp + k);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t a0[4], a1[4];
          ldsm4(a0, qp + m * 16 * pitch + k);
          ldsm4(a1, qp + m * 16 * pitch + k + 16);
          mma(c0[m], a0, bk[0], bk[1]);
          mma(c1[m], a1, bk[2], bk[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half)
          *reinterpret_cast<float2*>(sS + (m * 16 + lr + half * 8) * kSP + warp * 8 + lc) =
              make_float2((c0[m][half * 2] + c1[m][half * 2]) * sc, (c0[m][half * 2 + 1] + c1[m][half * 2 + 1]) * sc);
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m) {  // 16 lanes per head, 4 keys each
      const int r = m * 16 + (tid >> 4), c = (tid & 15) * 4;
      const float4 s4 = *reinterpret_cast<const float4*>(sS + r * kSP + c);
      float s[4] = {s4.x, s4.y, s4.z, s4.w};
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (j0 + c + i >= j_hi) s[i] = -INFINITY;
        mx = fmaxf(mx, s[i]);
      }
      for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float old = s_m[r], now = fmaxf(old, mx);  // every block has a visible key: now is finite
      float p[4], sum = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        p[i] = exp2f(s[i] - now);
        sum += p[i];
      }
      *reinterpret_cast<uint2*>(sP + r * kPP + c) = make_uint2(pack2(p[0], p[1]), pack2(p[2], p[3]));
      for (int off = 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      __syncwarp();
      if ((tid & 15) == 0) {
        const float alpha = exp2f(old - now);
        s_m[r] = now;
        s_alpha[r] = alpha;
        s_l[r] = s_l[r] * alpha + sum;
      }
    }
    __syncthreads();
    uint32_t ap[MT][4][4];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float al0 = s_alpha[m * 16 + lr], al1 = s_alpha[m * 16 + lr + 8];
#pragma unroll
      for (int i = 0; i < kLdMaxPairs; ++i)
#pragma unroll
        for (int u = 0; u < 2; ++u)
          acc[m][i][u][0] *= al0, acc[m][i][u][1] *= al0, acc[m][i][u][2] *= al1, acc[m][i][u][3] *= al1;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) ldsm4(ap[m][kk], sP + (m * 16 + (lane & 15)) * kPP + kk * 16 + (lane >> 4) * 8);
    }
#pragma unroll
    for (int i = 0; i < kLdMaxPairs; ++i) {
      const int pair = warp + i * kLdWarps;
      if (pair < n_pairs) {
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          uint32_t bv[4];
          ldsm4t(bv, sK + (kk * 16 + (lane & 15)) * pitch + pair * 16 + (lane >> 4) * 8);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma(acc[m][i][0], ap[m][kk], bv[0], bv[1]);
            mma(acc[m][i][1], ap[m][kk], bv[2], bv[3]);
          }
        }
      }
    }
    __syncthreads();  // the stage may be overwritten
  }
  cp_wait_all();
  __syncthreads();

  const int64_t first = (row * a.heads + h0) * a.splits + split;  // this split of the CTA's first head
  float* part = a.splits > 1 ? a.part + first * a.rot_off : nullptr;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < kLdMaxPairs; ++i) {
      const int pair = warp + i * kLdWarps;
      if (pair >= n_pairs) continue;
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = m * 16 + lr + half * 8, c = pair * 16 + u * 8 + lc;
          if (r < nh && c < a.rot_off) {  // rot_off is a multiple of 8
            const float x = acc[m][i][u][half * 2], y = acc[m][i][u][half * 2 + 1];
            if (part != nullptr) {
              *reinterpret_cast<float2*>(part + static_cast<int64_t>(r) * a.splits * a.rot_off + c) = make_float2(x, y);
            } else {
              const float inv = 1.f / s_l[r];
              *reinterpret_cast<uint32_t*>(out + r * a.out_ld + c) = pack2(x * inv, y * inv);
            }
          }
        }
    }
  if (part != nullptr && tid < nh)
    *reinterpret_cast<float2*>(a.part_ml + (first + static_cast<int64_t>(tid) * a.splits) * 2) = make_float2(s_m[tid], s_l[tid]);
}

// One CTA per (query row, head): parts weighted by their maxima, four columns per thread.
__global__ void __launch_bounds__(128) latent_merge_kernel(LatentArgs a) {
  __shared__ float s_w[kLdMaxSplits];
  const int64_t row = blockIdx.x;
  const int h = blockIdx.y, tid = threadIdx.x;
  if (token_position(a, static_cast<int>(row / a.T), static_cast<int>(row % a.T)) < 0) return;
  const int64_t first = (row * a.heads + h) * a.splits;
  if (tid < 32) {
    float m[kLdMaxSplits / 32], l[kLdMaxSplits / 32], mx = -INFINITY, total = 0.f;
#pragma unroll
    for (int i = 0; i < kLdMaxSplits / 32; ++i) {
      m[i] = -INFINITY, l[i] = 0.f;
      if (tid + i * 32 < a.splits) {
        const float2 ml = *reinterpret_cast<const float2*>(a.part_ml + (first + tid + i * 32) * 2);
        m[i] = ml.x, l[i] = ml.y;
      }
      mx = fmaxf(mx, m[i]);
    }
    for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
#pragma unroll
    for (int i = 0; i < kLdMaxSplits / 32; ++i) {
      m[i] = exp2f(m[i] - mx);  // a split without keys weighs 0
      total += m[i] * l[i];
    }
    for (int off = 16; off > 0; off >>= 1) total += __shfl_xor_sync(0xffffffffu, total, off);
#pragma unroll
    for (int i = 0; i < kLdMaxSplits / 32; ++i)
      if (tid + i * 32 < a.splits) s_w[tid + i * 32] = m[i] / total;
  }
  __syncthreads();
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (row * a.heads + h) * a.out_ld;
  for (int c = tid * 4; c < a.rot_off; c += 128 * 4) {
    const float* p = a.part + first * a.rot_off + c;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < a.splits; ++s) {
      const float4 v = *reinterpret_cast<const float4*>(p + static_cast<int64_t>(s) * a.rot_off);
      const float w = s_w[s];
      x.x += w * v.x, x.y += w * v.y, x.z += w * v.z, x.w += w * v.w;
    }
    *reinterpret_cast<uint2*>(out + c) = make_uint2(pack2(x.x, x.y), pack2(x.z, x.w));
  }
}

namespace {

int latent_launched() { return cudaGetLastError() == cudaSuccess ? 0 : -4; }

bool latent_bad(const LatentArgs& a) {
  return a.B <= 0 || a.T <= 0 || a.heads <= 0 || a.dim <= 0 || a.rot_dim <= 0 || a.rank <= 0 || a.slots <= 0 ||
         a.rot_dims < 0 || a.rot_dims % 2 || a.rot_dims > a.rot_dim || a.rot_off < a.rank || a.rot_off % 8 || a.row_w % 8 ||
         a.row_w < a.rot_off + a.rot_dim || a.cache_ld < a.row_w || a.B > 65535;
}

template <int MT>
int launch_latent_decode(const LatentArgs& a, cudaStream_t stream) {
  const int smem = ld_smem(a.row_w, MT * 16).total;
  static int configured = 48 * 1024;
  if (smem > configured) {
    if (smem > 227 * 1024 || cudaFuncSetAttribute(latent_decode_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                  smem) != cudaSuccess)
      return -3;
    configured = smem;
  }
  const dim3 grid(a.B * a.T, a.splits, (a.heads + MT * 16 - 1) / (MT * 16));
  latent_decode_kernel<MT><<<grid, kLdThreads, smem, stream>>>(a);
  if (a.splits > 1) latent_merge_kernel<<<dim3(a.B * a.T, a.heads), 128, 0, stream>>>(a);
  return latent_launched();
}

}  // namespace
}  // namespace axb

extern "C" int axb_latent_prep(const axb::LatentArgs* args, cudaStream_t stream) {
  const axb::LatentArgs& a = *args;
  if (axb::latent_bad(a)) return -10;
  const size_t smem = sizeof(float2) * (a.rot_dims / 2);
  if (smem > 48 * 1024) return -10;
  const int aligned = a.ld | a.cache_ld | a.lat_ld | a.dim | a.rot_dim | a.rank | a.q_off | a.c_off | a.r_off;
  if (a.act_bf16 && a.qbuf == nullptr && a.lat != nullptr && !(aligned & 7)) {
    const int64_t ctas = (static_cast<int64_t>(a.B) * a.T + axb::kLvTokens - 1) / axb::kLvTokens;
    if (smem * axb::kLvTokens <= 48 * 1024) {
      axb::latent_prep_vec_kernel<<<static_cast<unsigned>(ctas), 64 * axb::kLvTokens, smem * axb::kLvTokens, stream>>>(a);
      return axb::latent_launched();
    }
  }
  // Few tokens: the heads side by side; many: fewer copies of the trigonometry.
  const int heads_per = static_cast<int64_t>(a.B) * a.T <= 1024 ? 4 : 32;
  const dim3 grid(a.T, a.B, 1 + (a.heads + heads_per - 1) / heads_per);
  if (a.act_bf16)
    axb::latent_prep_kernel<__nv_bfloat16><<<grid, axb::kLpThreads, smem, stream>>>(a, heads_per);
  else
    axb::latent_prep_kernel<float><<<grid, axb::kLpThreads, smem, stream>>>(a, heads_per);
  return axb::latent_launched();
}

// rank <= 2048.
extern "C" int axb_latent_attn(const axb::LatentArgs* args, cudaStream_t stream) {
  const axb::LatentArgs& a = *args;
  const size_t smem = sizeof(float) * a.row_w;
  if (axb::latent_bad(a) || a.qbuf == nullptr || a.rot_off > axb::kLaThreads * axb::kLaCols || smem > 40 * 1024 ||
      a.heads > 65535 || static_cast<int64_t>(a.B) * a.T > 0x7fffffff)
    return -10;
  const dim3 grid(a.B * a.T, a.heads);
  if (a.act_bf16)
    axb::latent_attn_kernel<__nv_bfloat16><<<grid, axb::kLaThreads, smem, stream>>>(a);
  else
    axb::latent_attn_kernel<float><<<grid, axb::kLaThreads, smem, stream>>>(a);
  return axb::latent_launched();
}

// Whether the tensor-core kernel takes these sizes.
extern "C" int axb_latent_decode_supported(int row_w, int rank) {
  return rank <= 16 * axb::kLdWarps * axb::kLdMaxPairs && axb::ld_smem(row_w, 32).total <= 227 * 1024;
}

// bf16; splits > 1 needs part and part_ml.
extern "C" int axb_latent_decode(const axb::LatentArgs* args, cudaStream_t stream) {
  const axb::LatentArgs& a = *args;
  if (axb::latent_bad(a) || !a.act_bf16 || a.qbuf == nullptr || !axb_latent_decode_supported(a.row_w, a.rank) ||
      a.splits < 1 || a.splits > axb::kLdMaxSplits || a.cache_ld % 8 || a.out_ld % 8 || a.out_ld < a.rot_off ||
      a.heads > 65535 || static_cast<int64_t>(a.B) * a.T > 0x7fffffff)
    return -10;
  if (a.splits > 1 && (a.part == nullptr || a.part_ml == nullptr)) return -11;
  return a.heads > 16 ? axb::launch_latent_decode<2>(a, stream) : axb::launch_latent_decode<1>(a, stream);
}
