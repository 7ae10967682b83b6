// Softmax attention whose keys and values are projections of one cached latent per token (and, optionally, a rotated key
// part all heads share).  A cache row is [latent (rank), zeros to rank_pad, rotated part, zeros to width].
//
// Row by row (decoding, batches, f32 sessions, short portions) keys and values are never formed:
//   in     latent norm, rotation, cache row; the query against the key rows of its head: q . (U c) = (U^T q) . c
//   attn   per key range and eight heads: scores, online softmax, weighted latents
//   out    ranges merged, value rows of the head times the weighted latent, output gate
//
// Prompts form keys and values of the visible positions once (one product with the stacked key and value rows) and run an
// online-softmax kernel on the tensor cores (mma.sync bf16), 128 queries of a head per block.  Scores and weights are f32;
// the weights meet the values as two bf16 operands, high part and remainder.
#include <math.h>

#include "act.cuh"
#include "common.cuh"
#include "layered.h"
#include "mma_bf16.cuh"

namespace emelb {
namespace {

constexpr int kThreads = 128;
constexpr int kHG = 8;          // heads per block of the attention launch
constexpr int kKeys = 64;       // most keys per tile
constexpr int kCols = 512;      // latent columns per block of the attention launch
constexpr int kSlice = 64;      // latent columns per block of the query launch
constexpr int kOutTile = 32;    // values per block of the out launch
constexpr int kOutThreads = 512, kOutGroups = 4, kOutCols = 4 * kOutThreads / kOutGroups;   // a group adds up every fourth range
constexpr int kMaxSplits = 32;

__device__ __forceinline__ float from(float x) { return x; }
__device__ __forceinline__ float from(__nv_bfloat16 x) { return __bfloat162float(x); }
template <class T> __device__ __forceinline__ T to(float x);
template <> __device__ __forceinline__ float to<float>(float x) { return x; }
template <> __device__ __forceinline__ __nv_bfloat16 to<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }

__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const float2 a = unpack2(v.x), b = unpack2(v.y), c = unpack2(v.z), d = unpack2(v.w);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
}
__device__ __forceinline__ void load4(const float* p, float (&f)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&f)[4]) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack2(v.x), b = unpack2(v.y);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}

__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

__device__ __forceinline__ int row_pos(const Rows& r, int i) { return r.prompt ? r.pos[0] + i : r.pos[i]; }
__device__ __forceinline__ int row_seq(const Rows& r, int i) { return r.prompt ? r.seq0 : r.seq0 + i; }
__device__ __forceinline__ int first_key(int pos, int window) { return window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0; }

// pair p of a rotated vector of n dimensions: its two places
__device__ __forceinline__ void pair_of(int p, int n, int half, int& i, int& j) {
  i = half ? p : 2 * p;
  j = half ? p + n / 2 : 2 * p + 1;
}

// one block: the cache row of row r
template <class TC>
__device__ void store_latent(const LatentArgs& a, int r, int pos, int seq) {
  __shared__ float scratch[kThreads / 32];
  const float* x = a.down + (int64_t)r * a.ldd;
  TC* row = static_cast<TC*>(a.cache) + ((int64_t)seq * a.capacity + pos) * a.width;
  float ss = 0.0f;
  for (int i = threadIdx.x; i < a.rank; i += kThreads) ss = fmaf(x[i], x[i], ss);
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = ss;
  __syncthreads();
  const float inv = 1.0f / sqrtf((scratch[0] + scratch[1] + scratch[2] + scratch[3]) / a.rank + a.eps);
  for (int i = threadIdx.x; i < a.rank_pad; i += kThreads) row[i] = to<TC>(i < a.rank ? x[i] * inv * a.norm[i] : 0.0f);
  const float* k = x + a.rank;
  for (int p = threadIdx.x; p < a.rot / 2; p += kThreads) {
    int i, j;
    pair_of(p, a.rot, a.rope_half, i, j);
    const float c = a.rope_cos[(int64_t)pos * (a.rot / 2) + p], s = a.rope_sin[(int64_t)pos * (a.rot / 2) + p];
    row[a.rank_pad + i] = to<TC>(k[i] * c - k[j] * s);
    row[a.rank_pad + j] = to<TC>(k[j] * c + k[i] * s);
  }
  for (int i = a.rank_pad + a.rot + threadIdx.x; i < a.width; i += kThreads) row[i] = to<TC>(0.0f);
}

// grid (rows): cache row, and the row's queries rotated in place
__global__ void __launch_bounds__(kThreads) latent_store_kernel(const LatentArgs a, const Rows rows) {
  const int r = blockIdx.x, pos = row_pos(rows, r), pairs = a.rot / 2;
  store_latent<__nv_bfloat16>(a, r, pos, row_seq(rows, r));
  __nv_bfloat16* q = static_cast<__nv_bfloat16*>(a.proj) + (int64_t)r * a.ldp + a.dim;
  for (int x = threadIdx.x; x < a.heads * pairs; x += kThreads) {
    const int h = x / pairs, p = x - h * pairs;
    int i, j;
    pair_of(p, a.rot, a.rope_half, i, j);
    const float c = a.rope_cos[(int64_t)pos * pairs + p], s = a.rope_sin[(int64_t)pos * pairs + p];
    __nv_bfloat16* head = q + h * (a.dim + a.rot);
    const float u = from(head[i]), v = from(head[j]);
    head[i] = to<__nv_bfloat16>(u * c - v * s);
    head[j] = to<__nv_bfloat16>(v * c + u * s);
  }
}

// grid (column slices + 1, heads, rows): slices of U^T q of one head; the last slice rotates the head's query and, for
// head 0, stores the cache row
template <class TC, class TP>
__global__ void __launch_bounds__(kThreads) latent_in_kernel(const LatentArgs a, const Rows rows, int row0) {
  extern __shared__ float qs[];            // [dim], then the warps' partial columns
  pdl_trigger();
  const int h = blockIdx.y, r = row0 + blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (blockIdx.x < gridDim.x - 1)
    for (int d = tid; d < a.dim; d += kThreads) prefetch_l2(a.up.w + (int64_t)(h * a.dim + d) * a.up.ld + blockIdx.x * kSlice);
  pdl_wait();
  const TP* q = static_cast<const TP*>(a.proj) + (int64_t)r * a.ldp + h * (a.dim + a.rot);
  float* out = a.qlat + ((int64_t)blockIdx.z * a.heads + h) * a.width;
  if (blockIdx.x == gridDim.x - 1) {
    const int pos = row_pos(rows, r);
    for (int p = tid; p < a.rot / 2; p += kThreads) {
      int i, j;
      pair_of(p, a.rot, a.rope_half, i, j);
      const float c = a.rope_cos[(int64_t)pos * (a.rot / 2) + p], s = a.rope_sin[(int64_t)pos * (a.rot / 2) + p];
      const float u = from(q[a.dim + i]), v = from(q[a.dim + j]);
      out[a.rank_pad + i] = u * c - v * s;
      out[a.rank_pad + j] = v * c + u * s;
    }
    for (int i = a.rank_pad + a.rot + tid; i < a.width; i += kThreads) out[i] = 0.0f;
    if (h == 0) store_latent<TC>(a, r, pos, row_seq(rows, r));
    return;
  }
  float* part = qs + a.dim;                // [warps][kSlice]
  for (int i = tid; i < a.dim; i += kThreads) qs[i] = from(q[i]);
  __syncthreads();
  const int c = blockIdx.x * kSlice + 2 * lane;   // two columns per lane; rows of `up` are readable to a multiple of 8
  float s0 = 0.0f, s1 = 0.0f;
  if (c < a.rank_pad) {
    const __nv_bfloat16* w = a.up.w + (int64_t)h * a.dim * a.up.ld + c;
#pragma unroll 8
    for (int d = warp; d < a.dim; d += kThreads / 32) {
      const float2 x = unpack2(*reinterpret_cast<const uint32_t*>(w + (int64_t)d * a.up.ld));
      s0 = fmaf(qs[d], x.x, s0);
      s1 = fmaf(qs[d], x.y, s1);
    }
  }
  part[warp * kSlice + 2 * lane] = s0;
  part[warp * kSlice + 2 * lane + 1] = s1;
  __syncthreads();
  const int col = blockIdx.x * kSlice + tid;
  if (tid < kSlice && col < a.rank_pad) {
    float s = 0.0f;
#pragma unroll
    for (int w = 0; w < kThreads / 32; ++w) s += part[w * kSlice + tid];
    out[col] = col < a.rank ? s : 0.0f;
  }
}

// sums of N = 32 values over the warp's lanes; lane i returns with the sum of value i
__device__ __forceinline__ float transpose_sum(float (&v)[32]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float give = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  return v[0];
}

// grid (ranges x column blocks, head groups, rows); tiles of `keys` cache rows pass through shared memory
template <class TC>
__global__ void __launch_bounds__(kThreads) latent_attn_kernel(const LatentArgs a, const Rows rows, int row0, int splits, int keys) {
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;                          // [kHG][width]
  float* p = qs + kHG * a.width;           // [kHG][kKeys] scores, then weights
  TC* tile = reinterpret_cast<TC*>(p + kHG * kKeys);   // [keys][width]
  __shared__ float m_run[kHG], l_run[kHG], fix[kHG];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x % splits, col0 = blockIdx.x / splits * kCols, h0 = blockIdx.y * kHG, r = row0 + blockIdx.z;
  const int pos = row_pos(rows, r), lo = first_key(pos, a.window), n = pos - lo + 1;
  const int L = (n + splits - 1) / splits, k0 = min(n, split * L), k1 = min(n, k0 + L);
  const TC* cache = static_cast<const TC*>(a.cache) + ((int64_t)row_seq(rows, r) * a.capacity + lo) * a.width;
  constexpr int kPer16 = 16 / sizeof(TC);
  auto fetch = [&](int t0) {
    const TC* src = cache + (int64_t)t0 * a.width;
    for (int i = tid; i < min(keys, k1 - t0) * a.width / kPer16; i += kThreads) cp_async16(tile + i * kPer16, src + i * kPer16);
    cp_async_commit();
  };
  if (k0 < k1) fetch(k0);
  const float* q = a.qlat + ((int64_t)blockIdx.z * a.heads + h0) * a.width;
  for (int i = tid; i < kHG * a.width; i += kThreads) qs[i] = h0 + i / a.width < a.heads ? q[i] : 0.0f;
  if (tid < kHG) {
    m_run[tid] = -INFINITY;
    l_run[tid] = 0.0f;
  }
  const int col = col0 + 4 * tid;
  const bool mine = col < a.rank_pad;
  float acc[kHG][4] = {};
  for (int t0 = k0; t0 < k1; t0 += keys) {
    const int nt = min(keys, k1 - t0);
    cp_async_wait<0>();
    __syncthreads();
    // scores: four keys of a warp at a time, lanes across the row
    for (int kb = 4 * warp; kb < nt; kb += 4 * (kThreads / 32)) {
      const TC* kp[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) kp[u] = tile + min(kb + u, nt - 1) * a.width;
      float s[4 * kHG] = {};
      for (int c = 8 * lane; c < a.width; c += 256) {
        float kf[4][8];
#pragma unroll
        for (int u = 0; u < 4; ++u) load8(kp[u] + c, kf[u]);
#pragma unroll
        for (int h = 0; h < kHG; ++h) {
          float qf[8];
          load8(qs + h * a.width + c, qf);
#pragma unroll
          for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int e = 0; e < 8; ++e) s[4 * h + u] = fmaf(qf[e], kf[u][e], s[4 * h + u]);
        }
      }
      const float sum = transpose_sum(s);
      if (kb + (lane & 3) < nt) p[(lane >> 2) * kKeys + kb + (lane & 3)] = sum * a.scale;
    }
    __syncthreads();
    for (int h = warp; h < kHG; h += kThreads / 32) {
      const float s0 = lane < nt ? p[h * kKeys + lane] : -INFINITY, s1 = lane + 32 < nt ? p[h * kKeys + lane + 32] : -INFINITY;
      float m = fmaxf(s0, s1);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      const float before = m_run[h];
      m = fmaxf(m, before);
      const float w0 = expf(s0 - m), w1 = expf(s1 - m);
      p[h * kKeys + lane] = w0;
      p[h * kKeys + lane + 32] = w1;
      const float l = warp_sum(w0 + w1), f = expf(before - m);
      if (lane == 0) {
        m_run[h] = m;
        l_run[h] = l_run[h] * f + l;
        fix[h] = f;
      }
    }
    __syncthreads();
    if (mine) {
#pragma unroll
      for (int h = 0; h < kHG; ++h)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[h][e] *= fix[h];
      for (int k = 0; k < nt; k += 4) {
        float v[4][4];
#pragma unroll
        for (int u = 0; u < 4; ++u) load4(tile + min(k + u, nt - 1) * a.width + col, v[u]);   // weights past nt are 0
#pragma unroll
        for (int h = 0; h < kHG; ++h) {
          const float4 w = *reinterpret_cast<const float4*>(p + h * kKeys + k);
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[h][e] = fmaf(w.w, v[3][e], fmaf(w.z, v[2][e], fmaf(w.y, v[1][e], fmaf(w.x, v[0][e], acc[h][e]))));
        }
      }
    }
    __syncthreads();
    if (t0 + keys < k1) fetch(t0 + keys);
  }
  __syncthreads();
  if (mine)
#pragma unroll
    for (int h = 0; h < kHG; ++h)
      if (h0 + h < a.heads)
        *reinterpret_cast<float4*>(a.part + (((int64_t)blockIdx.z * splits + split) * a.heads + h0 + h) * a.rank_pad + col) =
            make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]);
  if (col0 == 0 && tid < kHG && h0 + tid < a.heads)
    reinterpret_cast<float2*>(a.stats)[((int64_t)blockIdx.z * splits + split) * a.heads + h0 + tid] = make_float2(m_run[tid], l_run[tid]);
}

// grid (value tiles, heads, rows)
template <class TP, class TO>
__global__ void __launch_bounds__(kOutThreads) latent_out_kernel(const LatentArgs a, const Rows rows, int row0, int splits, TO* __restrict__ out, int64_t ldo) {
  extern __shared__ __align__(16) float o[];    // [rank_pad]
  __shared__ float4 sums[kOutGroups][kOutCols / 4];
  __shared__ float weight[kMaxSplits];
  pdl_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, r = row0 + blockIdx.z;
  const int e0 = blockIdx.x * kOutTile, e1 = min(a.vdim, e0 + kOutTile);
  const __nv_bfloat16* up = a.up.w + ((int64_t)a.heads * a.dim + (int64_t)h * a.vdim) * a.up.ld;
  for (int64_t c = 64 * tid; c < (e1 - e0) * a.up.ld; c += 64 * kOutThreads) prefetch_l2(up + e0 * a.up.ld + c);
  pdl_wait();
  const int group = tid / (kOutCols / 4), quad = tid % (kOutCols / 4);
  const float* part = a.part + ((int64_t)blockIdx.z * splits * a.heads + h) * a.rank_pad;
  const int64_t stride = (int64_t)a.heads * a.rank_pad;
  // the first columns' sums are requested before the ranges' weights are known
  float4 first[kMaxSplits / kOutGroups];
#pragma unroll
  for (int i = 0; i < kMaxSplits / kOutGroups; ++i) {
    const int s = group + kOutGroups * i;
    first[i] = s < splits && 4 * quad < a.rank_pad ? *reinterpret_cast<const float4*>(part + s * stride + 4 * quad) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  if (warp == 0) {
    const float2 s = lane < splits ? reinterpret_cast<const float2*>(a.stats)[((int64_t)blockIdx.z * splits + lane) * a.heads + h] : make_float2(-INFINITY, 0.0f);
    float m = s.x;
#pragma unroll
    for (int k = 16; k > 0; k >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, k));
    const float f = s.x > -INFINITY ? expf(s.x - m) : 0.0f;
    weight[lane] = f / warp_sum(f * s.y);
  }
  __syncthreads();
  for (int c0 = 0; c0 < a.rank_pad; c0 += kOutCols) {
    const int c = c0 + 4 * quad;
    float4 t = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < kMaxSplits / kOutGroups; ++i) {
      const int s = group + kOutGroups * i;
      if (s >= splits || c >= a.rank_pad) break;
      const float w = weight[s];
      const float4 v = c0 == 0 ? first[i] : *reinterpret_cast<const float4*>(part + s * stride + c);
      t.x = fmaf(w, v.x, t.x);
      t.y = fmaf(w, v.y, t.y);
      t.z = fmaf(w, v.z, t.z);
      t.w = fmaf(w, v.w, t.w);
    }
    sums[group][quad] = t;
    __syncthreads();
    for (int x = tid; x < min(kOutCols, a.rank_pad - c0); x += kOutThreads) {
      float v = 0.0f;
#pragma unroll
      for (int g = 0; g < kOutGroups; ++g) v += reinterpret_cast<const float*>(sums[g])[x];
      o[c0 + x] = v;
    }
    __syncthreads();
  }
  const TP* gate = a.gate_at ? static_cast<const TP*>(a.proj) + (int64_t)r * a.ldp + a.gate_at + h * a.vdim : nullptr;
#pragma unroll 2
  for (int e = e0 + warp; e < e1; e += kOutThreads / 32) {
    const __nv_bfloat16* w = up + (int64_t)e * a.up.ld;
    float s = 0.0f;
    for (int c = 8 * lane; c < a.rank_pad; c += 256) {
      float wf[8], of[8];
      load8(w + c, wf);
      load8(o + c, of);
#pragma unroll
      for (int i = 0; i < 8; ++i) s = fmaf(wf[i], of[i], s);
    }
    s = warp_sum(s);
    if (lane == 0) {
      if (gate) s *= sigmoidf_(from(gate[e]));
      out[(int64_t)r * ldo + h * a.vdim + e] = to<TO>(s);
    }
  }
}

// ---- the attention launch on the tensor cores (mma.sync bf16): bf16 caches with at most kMmaCols latent columns.  Sixteen
// heads per block are the rows of both products; query and weights are fed as two bf16 operands, high part and remainder.
constexpr int kMmaHeads = 16, kMmaThreads = 256, kMmaCols = 64 * kMmaThreads / 32;

struct MmaShape {
  int kw, row, smem;     // columns of the score product (a multiple of 16), elements between rows in shared memory
};
MmaShape mma_shape(const LatentArgs& a) {
  MmaShape s;
  s.kw = (a.width + 15) / 16 * 16;
  s.row = s.kw + 8;
  s.smem = 2 * (2 * kMmaHeads + kKeys) * s.row + 4 * kMmaHeads * (kKeys + 4) + 2 * 2 * kMmaHeads * (kKeys + 8) + 32;
  return s;
}

// grid (ranges, head groups, rows)
__global__ void __launch_bounds__(kMmaThreads) latent_attn_mma_kernel(const LatentArgs a, const Rows rows, int row0, int splits, const MmaShape shape) {
  extern __shared__ __align__(16) unsigned char raw[];
  constexpr int kPRow = kKeys + 8, kSRow = kKeys + 4;
  const int R = shape.row;
  __nv_bfloat16* q_hi = reinterpret_cast<__nv_bfloat16*>(raw);      // [kMmaHeads][R]
  __nv_bfloat16* q_lo = q_hi + kMmaHeads * R;
  __nv_bfloat16* tile = q_lo + kMmaHeads * R;                       // [kKeys][R]
  __nv_bfloat16* p_hi = tile + kKeys * R + 16;                      // [kMmaHeads][kPRow]  (a load of two column blocks may look past the last row)
  __nv_bfloat16* p_lo = p_hi + kMmaHeads * kPRow;
  float* sc = reinterpret_cast<float*>(p_lo + kMmaHeads * kPRow);   // [kMmaHeads][kSRow]
  __shared__ float m_run[kMmaHeads], l_run[kMmaHeads], fix[kMmaHeads];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int split = blockIdx.x, h0 = blockIdx.y * kMmaHeads, r = row0 + blockIdx.z;
  const int pos = row_pos(rows, r), lo = first_key(pos, a.window), n = pos - lo + 1;
  const int L = (n + splits - 1) / splits, k0 = min(n, split * L), k1 = min(n, k0 + L);
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(a.cache) + ((int64_t)row_seq(rows, r) * a.capacity + lo) * a.width;
  const int chunks = shape.kw / 8, live_chunks = a.width / 8;
  auto fetch = [&](int t0) {
    for (int i = tid; i < kKeys * chunks; i += kMmaThreads) {
      const int k = i / chunks, c = i - k * chunks;
      const bool live = t0 + k < k1 && c < live_chunks;
      cp16_zfill(tile + k * R + 8 * c, live ? cache + (int64_t)(t0 + k) * a.width + 8 * c : cache, live);
    }
    cp_async_commit();
  };
  if (k0 < k1) fetch(k0);
  const float* q = a.qlat + ((int64_t)blockIdx.z * a.heads + h0) * a.width;
  for (int i = tid; i < kMmaHeads * shape.kw / 2; i += kMmaThreads) {
    const int h = i / (shape.kw / 2), c = i % (shape.kw / 2) * 2;
    const float2 v = h0 + h < a.heads && c < a.width ? *reinterpret_cast<const float2*>(q + (int64_t)h * a.width + c) : make_float2(0.0f, 0.0f);
    uint32_t hi, rest;
    split2(v.x, v.y, hi, rest);
    *reinterpret_cast<uint32_t*>(q_hi + h * R + c) = hi;
    *reinterpret_cast<uint32_t*>(q_lo + h * R + c) = rest;
  }
  if (tid < kMmaHeads) {
    m_run[tid] = -INFINITY;
    l_run[tid] = 0.0f;
  }
  float acc[8][4] = {};
  const int c0 = 64 * warp;
  for (int t0 = k0; t0 < k1; t0 += kKeys) {
    const int nt = min(kKeys, k1 - t0);
    cp_async_wait<0>();
    __syncthreads();
    {
      // eight keys per warp
      float s[2][4] = {};
      const __nv_bfloat16* kb = tile + (8 * warp + (lane & 7)) * R + 8 * (lane >> 3);
      const int qa = (lane & 15) * R + (lane >> 4) * 8;
#pragma unroll 3
      for (int d = 0; d < shape.kw; d += 32) {
        uint32_t b[4], x[4];
        ldsm(b, kb + d);
        ldsm(x, q_hi + qa + d);
        mma_bf16_16816(s[0], x, b[0], b[1]);
        ldsm(x, q_lo + qa + d);
        mma_bf16_16816(s[1], x, b[0], b[1]);
        if (d + 16 < shape.kw) {
          ldsm(x, q_hi + qa + d + 16);
          mma_bf16_16816(s[0], x, b[2], b[3]);
          ldsm(x, q_lo + qa + d + 16);
          mma_bf16_16816(s[1], x, b[2], b[3]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) sc[(g + 8 * (e >> 1)) * kSRow + 8 * warp + 2 * t + (e & 1)] = (s[0][e] + s[1][e]) * a.scale;
    }
    __syncthreads();
    for (int h = warp; h < kMmaHeads; h += kMmaThreads / 32) {
      const float s0 = 2 * lane < nt ? sc[h * kSRow + 2 * lane] : -INFINITY, s1 = 2 * lane + 1 < nt ? sc[h * kSRow + 2 * lane + 1] : -INFINITY;
      float m = fmaxf(s0, s1);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      const float before = m_run[h];
      m = fmaxf(m, before);
      const float w0 = expf(s0 - m), w1 = expf(s1 - m);
      uint32_t hi, rest;
      split2(w0, w1, hi, rest);
      *reinterpret_cast<uint32_t*>(p_hi + h * kPRow + 2 * lane) = hi;
      *reinterpret_cast<uint32_t*>(p_lo + h * kPRow + 2 * lane) = rest;
      const float l = warp_sum(w0 + w1), f = expf(before - m);
      if (lane == 0) {
        m_run[h] = m;
        l_run[h] = l_run[h] * f + l;
        fix[h] = f;
      }
    }
    __syncthreads();
    const float f0 = fix[g], f1 = fix[g + 8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      acc[i][0] *= f0;
      acc[i][1] *= f0;
      acc[i][2] *= f1;
      acc[i][3] *= f1;
    }
#pragma unroll
    for (int kk = 0; kk < kKeys / 16; ++kk) {
      if (16 * kk >= nt) break;
      uint32_t hi[4], rest[4];
      ldsm(hi, p_hi + (lane & 15) * kPRow + 16 * kk + (lane >> 4) * 8);
      ldsm(rest, p_lo + (lane & 15) * kPRow + 16 * kk + (lane >> 4) * 8);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        if (c0 + 16 * np >= a.rank_pad) break;
        uint32_t b[4];
        ldsm_trans(b, tile + (16 * kk + (lane & 15)) * R + c0 + 16 * np + (lane >> 4) * 8);
        mma_bf16_16816(acc[2 * np], hi, b[0], b[1]);
        mma_bf16_16816(acc[2 * np + 1], hi, b[2], b[3]);
        mma_bf16_16816(acc[2 * np], rest, b[0], b[1]);
        mma_bf16_16816(acc[2 * np + 1], rest, b[2], b[3]);
      }
    }
    __syncthreads();
    if (t0 + kKeys < k1) fetch(t0 + kKeys);
  }
  __syncthreads();
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int h = h0 + g + 8 * half;
    if (h >= a.heads) continue;
    float* dst = a.part + (((int64_t)blockIdx.z * splits + split) * a.heads + h) * a.rank_pad;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = c0 + 8 * i + 2 * t;
      if (c < a.rank_pad) *reinterpret_cast<float2*>(dst + c) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
    }
  }
  if (tid < kMmaHeads && h0 + tid < a.heads)
    reinterpret_cast<float2*>(a.stats)[((int64_t)blockIdx.z * splits + split) * a.heads + h0 + tid] = make_float2(m_run[tid], l_run[tid]);
}

}  // namespace

template <class TC, class TP, class TO>
cudaError_t launch_latent_rows(const LatentArgs& a, const Rows& rows, TO* out, int64_t ldo, int sm_count, bool pdl, cudaStream_t st, int* launches) {
  const MmaShape shape = mma_shape(a);
  const bool mma = sizeof(TC) == 2 && a.rank_pad <= kMmaCols && shape.smem <= 220 * 1024;
  const int per_group = mma ? kMmaHeads : kHG, groups = (a.heads + per_group - 1) / per_group, blocks = mma ? 1 : (a.rank_pad + kCols - 1) / kCols;
  // about one tile of keys per range at least, two blocks per SM at most
  int splits = 1;
  if (rows.n <= kLatentRows) {
    splits = (a.max_visible + kKeys - 1) / kKeys;
    const int fill = (2 * sm_count + groups * blocks - 1) / (groups * blocks);
    splits = splits > fill ? fill : splits;
    splits = splits > kMaxSplits ? kMaxSplits : splits;
  }
  const size_t s_in = 4 * ((size_t)a.dim + kThreads / 32 * kSlice), s_q = 4 * (size_t)kHG * (a.width + kKeys), s_out = 4 * (size_t)a.rank_pad;
  // two blocks per SM where a tile of 16 keys at least allows it
  int keys = kKeys;
  auto s_tile = [&](int k) { return s_q + sizeof(TC) * (size_t)k * a.width; };
  while (keys > 16 && s_tile(keys) > 110 * 1024) keys /= 2;
  while (keys > 1 && s_tile(keys) > 220 * 1024) keys /= 2;
  const size_t s_attn = s_tile(keys);
  if (s_in > 48 * 1024 || s_attn > 220 * 1024 || s_out > 200 * 1024) return cudaErrorInvalidValue;
  // the same limits for every size: launches of other sizes may already be in a captured step
  cudaError_t e = cudaFuncSetAttribute(latent_attn_kernel<TC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(latent_attn_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(latent_out_kernel<TP, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  if (e != cudaSuccess) return e;
  uint64_t fit = kLatentRows;
  const uint64_t per_part = (uint64_t)splits * a.heads * a.rank_pad, per_stats = 2ull * splits * a.heads;
  if (a.part_floats / per_part < fit) fit = a.part_floats / per_part;
  if (a.stats_floats / per_stats < fit) fit = a.stats_floats / per_stats;
  if (fit < 1) return cudaErrorInvalidValue;
  for (int r0 = 0; r0 < rows.n; r0 += (int)fit) {
    const int n = rows.n - r0 < (int)fit ? rows.n - r0 : (int)fit;
    e = launch_kernel(latent_in_kernel<TC, TP>, dim3((a.rank_pad + kSlice - 1) / kSlice + 1, a.heads, n), dim3(kThreads), s_in, st, pdl, a, rows, r0);
    if (e == cudaSuccess) {
      if (mma) e = launch_kernel(latent_attn_mma_kernel, dim3(splits, groups, n), dim3(kMmaThreads), (size_t)shape.smem, st, pdl, a, rows, r0, splits, shape);
      else e = launch_kernel(latent_attn_kernel<TC>, dim3(splits * blocks, groups, n), dim3(kThreads), s_attn, st, pdl, a, rows, r0, splits, keys);
    }
    if (e == cudaSuccess)
      e = launch_kernel(latent_out_kernel<TP, TO>, dim3((a.vdim + kOutTile - 1) / kOutTile, a.heads, n), dim3(kOutThreads), s_out, st, pdl, a, rows, r0, splits, out, ldo);
    if (e != cudaSuccess) return e;
    *launches += 3;
  }
  return cudaSuccess;
}
template cudaError_t launch_latent_rows<float, float, float>(const LatentArgs&, const Rows&, float*, int64_t, int, bool, cudaStream_t, int*);
template cudaError_t launch_latent_rows<__nv_bfloat16, float, float>(const LatentArgs&, const Rows&, float*, int64_t, int, bool, cudaStream_t, int*);
template cudaError_t launch_latent_rows<__nv_bfloat16, __nv_bfloat16, __nv_bfloat16>(const LatentArgs&, const Rows&, __nv_bfloat16*, int64_t, int, bool,
                                                                                     cudaStream_t, int*);

// ---- prompts
namespace {

constexpr int kQT = 128, kKT = 64, kPromptThreads = 256;
constexpr int kPromptMinRows = 9;   // fewer rows go through the latents: forming every visible key costs more

struct PromptShape {
  int qrow, vrow;          // elements between rows of the query / key and value tiles
  int smem;
};
PromptShape prompt_shape(const LatentArgs& a) {
  PromptShape s;
  s.qrow = (a.dim + a.rot + 15) / 16 * 16 + 8;
  s.vrow = (a.vdim + 15) / 16 * 16 + 8;
  s.smem = 2 * (kQT * s.qrow + 2 * kKT * (s.qrow + s.vrow));
  return s;
}

// grid (query tiles, heads).  NV: 8-column tiles of the values (vdim <= 8 NV).  key0: position of the first row of a.kv
template <int NV>
__global__ void __launch_bounds__(kPromptThreads) latent_prompt_kernel(const LatentArgs a, const Rows rows, const int key0, const PromptShape shape,
                                                                       __nv_bfloat16* __restrict__ out, int64_t ldo) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int QR = shape.qrow, VR = shape.vrow, D = a.dim + a.rot;
  __nv_bfloat16* qt = reinterpret_cast<__nv_bfloat16*>(raw);   // [kQT][QR]
  __nv_bfloat16* kt = qt + kQT * QR;                           // [2][kKT][QR]
  __nv_bfloat16* vt = kt + 2 * kKT * QR;                       // [2][kKT][VR]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int i0 = (gridDim.x - 1 - blockIdx.x) * kQT, h = blockIdx.y;   // tiles with the most keys first
  const int pos0 = rows.pos[0], last = min(rows.n, i0 + kQT) - 1;
  const int k_begin = first_key(pos0 + i0, a.window), k_end = pos0 + last + 1;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.proj) + (int64_t)i0 * a.ldp + h * D;
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(a.cache) + (int64_t)rows.seq0 * a.capacity * a.width + a.rank_pad;
  const __nv_bfloat16 *kb = a.kv + h * a.dim, *vb = a.kv + a.heads * a.dim + h * a.vdim;
  const int kc = (QR - 8) / 8, vc = (VR - 8) / 8, dc = a.dim / 8, xc = D / 8, vlive = a.vdim / 8;
  for (int i = tid; i < kQT * kc; i += kPromptThreads) {
    const int r = i / kc, c = i - r * kc;
    const bool live = i0 + r < rows.n && c < xc;
    cp16_zfill(qt + r * QR + 8 * c, live ? q + (int64_t)r * a.ldp + 8 * c : q, live);
  }
  auto issue = [&](int key, int buf) {
    for (int i = tid; i < kKT * kc; i += kPromptThreads) {
      const int r = i / kc, c = i - r * kc;
      const bool live = key + r < k_end && c < xc;
      const __nv_bfloat16* p = c < dc ? kb + (int64_t)(key + r - key0) * a.kv_ld + 8 * c : cache + (int64_t)(key + r) * a.width + 8 * (c - dc);
      cp16_zfill(kt + (buf * kKT + r) * QR + 8 * c, live ? p : a.kv, live);
    }
    for (int i = tid; i < kKT * vc; i += kPromptThreads) {
      const int r = i / vc, c = i - r * vc;
      const bool live = key + r < k_end && c < vlive;
      cp16_zfill(vt + (buf * kKT + r) * VR + 8 * c, live ? vb + (int64_t)(key + r - key0) * a.kv_ld + 8 * c : a.kv, live);
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  issue(k_begin, 0);

  float o[NV][4] = {};
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
  const float scale = a.scale * 1.4426950408889634f;   // weights as powers of two
  const int row0 = i0 + 16 * warp, p_lo = pos0 + row0;   // this warp's first query
  int buf = 0;
  for (int key = k_begin; key < k_end; key += kKT, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();   // the tile has landed, the other buffer is free
    if (key + kKT < k_end) issue(key + kKT, buf ^ 1);
    // nothing of the tile is visible to the warp's rows
    if (row0 >= rows.n || key > p_lo + 15 || key + kKT <= first_key(p_lo, a.window)) continue;
    const __nv_bfloat16 *kk = kt + buf * kKT * QR, *vv = vt + buf * kKT * VR;
    float s[kKT / 8][4] = {};
#pragma unroll 4
    for (int d = 0; d < QR - 8; d += 16) {
      uint32_t qa[4];
      ldsm(qa, qt + (16 * warp + (lane & 15)) * QR + d + (lane >> 4) * 8);
#pragma unroll
      for (int nt = 0; nt < kKT / 16; ++nt) {
        uint32_t b[4];
        ldsm(b, kk + (16 * nt + (lane & 7) + (lane >> 4) * 8) * QR + d + ((lane >> 3) & 1) * 8);
        mma_bf16_16816(s[2 * nt], qa, b[0], b[1]);
        mma_bf16_16816(s[2 * nt + 1], qa, b[2], b[3]);
      }
    }
    const bool inside = key + kKT - 1 <= p_lo && key >= first_key(p_lo + 15, a.window);
    float fix[2];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int pos = p_lo + g + 8 * half, lo = first_key(pos, a.window);
      float mx = m[half];
#pragma unroll
      for (int nt = 0; nt < kKT / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float& x = s[nt][2 * half + e];
          const int k = key + 8 * nt + 2 * t + e;
          x = inside || (k <= pos && k >= lo) ? x * scale : -INFINITY;
          mx = fmaxf(mx, x);
        }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));   // the four lanes of a row
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float base = mx == -INFINITY ? 0.0f : mx;
      fix[half] = exp2f(m[half] - base);
      m[half] = mx;
      float sum = 0.0f;
#pragma unroll
      for (int nt = 0; nt < kKT / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float& x = s[nt][2 * half + e];
          x = exp2f(x - base);
          sum += x;
        }
      l[half] = l[half] * fix[half] + sum;   // this lane's columns
    }
#pragma unroll
    for (int nv = 0; nv < NV; ++nv)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[nv][e] *= fix[e >> 1];
#pragma unroll
    for (int k16 = 0; k16 < kKT / 16; ++k16) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int part = 0; part < 2; ++part)
#pragma unroll
        for (int half = 0; half < 2; ++half) split2(s[2 * k16 + part][2 * half], s[2 * k16 + part][2 * half + 1], hi[2 * part + half], lo[2 * part + half]);
#pragma unroll
      for (int np = 0; np < NV / 2; ++np) {
        if (16 * np >= a.vdim) break;
        uint32_t b[4];
        ldsm_trans(b, vv + (16 * k16 + (lane & 15)) * VR + 16 * np + (lane >> 4) * 8);
        mma_bf16_16816(o[2 * np], hi, b[0], b[1]);
        mma_bf16_16816(o[2 * np + 1], hi, b[2], b[3]);
        mma_bf16_16816(o[2 * np], lo, b[0], b[1]);
        mma_bf16_16816(o[2 * np + 1], lo, b[2], b[3]);
      }
    }
  }
  const __nv_bfloat16* gate = a.gate_at ? static_cast<const __nv_bfloat16*>(a.proj) + a.gate_at + h * a.vdim : nullptr;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    float sum = l[half];
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    const int r = row0 + g + 8 * half;
    if (r >= rows.n) continue;
    const float inv = 1.0f / sum;
    __nv_bfloat16* dst = out + (int64_t)r * ldo + h * a.vdim;
#pragma unroll
    for (int nv = 0; nv < NV; ++nv) {
      const int c = 8 * nv + 2 * t;
      if (c >= a.vdim) continue;
      float x = o[nv][2 * half] * inv, y = o[nv][2 * half + 1] * inv;
      if (gate) {
        const float2 z = unpack2(*reinterpret_cast<const uint32_t*>(gate + (int64_t)r * a.ldp + c));
        x *= sigmoidf_(z.x);
        y *= sigmoidf_(z.y);
      }
      *reinterpret_cast<__nv_bfloat162*>(dst + c) = __floats2bfloat162_rn(x, y);
    }
  }
}

template <int NV>
cudaError_t launch_prompt_tiles(const LatentArgs& a, const Rows& rows, int key0, __nv_bfloat16* out, int64_t ldo, cudaStream_t st) {
  const PromptShape s = prompt_shape(a);
  const cudaError_t e = cudaFuncSetAttribute(latent_prompt_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, s.smem);
  if (e != cudaSuccess) return e;
  latent_prompt_kernel<NV><<<dim3((rows.n + kQT - 1) / kQT, a.heads), kPromptThreads, s.smem, st>>>(a, rows, key0, s, out, ldo);
  return cudaGetLastError();
}

}  // namespace

bool latent_prompt_supported(const LatentArgs& a, int rows) {
  return rows >= kPromptMinRows && a.dim % 8 == 0 && a.rot % 8 == 0 && a.vdim % 8 == 0 && a.vdim <= 256 && a.dim + a.rot <= 256 && a.ldp % 8 == 0 && a.kv &&
         prompt_shape(a).smem <= 227 * 1024;
}

cudaError_t launch_latent_prompt(const LatentArgs& a, const TmaMap& upmap, const Rows& rows, int pos0, __nv_bfloat16* out, int64_t ldo, int* status,
                                 cudaStream_t st, int* launches) {
  latent_store_kernel<<<rows.n, kThreads, 0, st>>>(a, rows);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return e;
  const int key0 = a.window > 0 && pos0 - a.window + 1 > 0 ? pos0 - a.window + 1 : 0, keys = pos0 + rows.n - key0;
  if (keys > a.kv_rows) return cudaErrorInvalidValue;
  // keys and values of the visible positions
  const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(a.cache) + ((int64_t)rows.seq0 * a.capacity + key0) * a.width;
  XMaps x;
  if (!encode_bf16_map(&x.narrow, base, keys, a.rank, a.width, kGemmTokenBox) || !encode_bf16_map(&x.wide, base, keys, a.rank, a.width, 128))
    return cudaErrorInvalidValue;
  e = launch_gemm_bf16(LinearArgs{a.up, nullptr, ACT_NONE, 0, keys}, upmap, x, nullptr, a.kv, a.kv_ld, status, st);
  if (e != cudaSuccess) return e;
  if (a.vdim <= 32) e = launch_prompt_tiles<4>(a, rows, key0, out, ldo, st);
  else if (a.vdim <= 64) e = launch_prompt_tiles<8>(a, rows, key0, out, ldo, st);
  else if (a.vdim <= 128) e = launch_prompt_tiles<16>(a, rows, key0, out, ldo, st);
  else e = launch_prompt_tiles<32>(a, rows, key0, out, ldo, st);
  *launches += 3;
  return e;
}

}  // namespace emelb
