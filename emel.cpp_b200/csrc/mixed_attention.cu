// Softmax attention over a sliding window that keeps the sequence's first tokens, with the heads' weights mixed after
// the softmax: weight_h <- sum_g talk[h][g] weight_g, head h then weighs its own key/value head's rows.
//
// A head's output needs every head's normalised weights, so scores and weighted sum are separate launches:
//   scores   raw scaled scores of each (row, head) over the visible keys, and {max, sum of exponentials} per key range
//   values   per key range and key/value head: all heads' weights from the scores, the mixed weights of that group's
//            heads, and their partial sums over the value rows
//   reduce   partial sums of the ranges added in order
// Visible keys of position i, in order: the kept tokens below the window (0 .. kk-1), then the window (lo .. i).
#include <math.h>

#include "common.cuh"
#include "layered.h"
#include "mma_bf16.cuh"

namespace emelb {
namespace {

constexpr int kThreads = 128;
constexpr int kTileKeys = 64;
constexpr int kMaxNRep = 8;

struct Span {
  int lo, kk, n;
  __device__ __forceinline__ int key(int idx) const { return idx < kk ? idx : lo + idx - kk; }
};
__device__ __forceinline__ Span span_of(int pos, int window, int keep) {
  Span s;
  s.lo = window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0;
  s.kk = keep < s.lo ? keep : s.lo;
  s.n = s.kk + pos - s.lo + 1;
  return s;
}

__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const uint32_t q[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(q[i] << 16);
    f[2 * i + 1] = __uint_as_float(q[i] & 0xffff0000u);
  }
}

template <class T> __device__ __forceinline__ T to(float x);
template <> __device__ __forceinline__ float to<float>(float x) { return x; }
template <> __device__ __forceinline__ __nv_bfloat16 to<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }

__device__ __forceinline__ int row_pos(const Rows& r, int i) { return r.prompt ? r.pos[0] + i : r.pos[i]; }
__device__ __forceinline__ int row_seq(const Rows& r, int i) { return r.prompt ? r.seq0 : r.seq0 + i; }

// grid (ranges, kv heads, rows).  Eight lanes per key, KU keys per lane group at a time, NR query heads at a time.
template <class T, int NR>
__global__ void __launch_bounds__(kThreads) mix_scores_kernel(const MixAttnArgs a, const Rows rows, int row0, int splits, int stride) {
  extern __shared__ __align__(16) float qs[];   // [n_rep][dim_pad]
  __shared__ float red[2][kMaxNRep][4];
  constexpr int KU = 4;
  const int tid = threadIdx.x, l8 = tid & 7, slot = tid >> 3;
  const int split = blockIdx.x, g = blockIdx.y, row = row0 + blockIdx.z;
  const int n_rep = a.heads / a.kv_heads, D = a.dim_pad;
  const Span sp = span_of(row_pos(rows, row), a.window, a.keep_first);
  const int L = (sp.n + splits - 1) / splits, i0 = min(sp.n, split * L), i1 = min(sp.n, i0 + L);
  const T* q = static_cast<const T*>(a.q) + ((int64_t)row * a.heads + g * n_rep) * D;
  for (int i = tid * 8; i < n_rep * D; i += kThreads * 8) {
    float f[8];
    load8(q + i, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) qs[i + e] = f[e];
  }
  __syncthreads();
  const T* kbase = static_cast<const T*>(a.k) + ((int64_t)row_seq(rows, row) * a.kv_heads + g) * a.capacity * D;
  float* sc = a.scores + ((int64_t)blockIdx.z * a.heads + g * n_rep) * stride;
  float2* stats = reinterpret_cast<float2*>(a.stats) + ((int64_t)blockIdx.z * splits + split) * a.heads + g * n_rep;

  for (int h0 = 0; h0 < n_rep; h0 += NR) {
    float mx[NR];
#pragma unroll
    for (int r = 0; r < NR; ++r) mx[r] = -INFINITY;
    for (int ib = i0; ib < i1; ib += 16 * KU) {
      const T* kp[KU];
#pragma unroll
      for (int u = 0; u < KU; ++u) kp[u] = kbase + (int64_t)sp.key(min(ib + slot + 16 * u, i1 - 1)) * D;
      float acc[NR][KU] = {};
      for (int c = l8 * 8; c < D; c += 64) {
        float kf[KU][8];
#pragma unroll
        for (int u = 0; u < KU; ++u) load8(kp[u] + c, kf[u]);
#pragma unroll
        for (int r = 0; r < NR; ++r) {
          float qf[8];
          load8(qs + (h0 + r) * D + c, qf);
#pragma unroll
          for (int u = 0; u < KU; ++u)
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[r][u] = fmaf(qf[e], kf[u][e], acc[r][u]);
        }
      }
#pragma unroll
      for (int r = 0; r < NR; ++r)
#pragma unroll
        for (int u = 0; u < KU; ++u) {
          float s = acc[r][u];
          s += __shfl_xor_sync(0xffffffffu, s, 1);
          s += __shfl_xor_sync(0xffffffffu, s, 2);
          s += __shfl_xor_sync(0xffffffffu, s, 4);
          s *= a.scale;
          const int idx = ib + slot + 16 * u;
          if (idx < i1) {
            mx[r] = fmaxf(mx[r], s);
            if (l8 == 0) sc[(int64_t)(h0 + r) * stride + idx] = s;
          }
        }
    }
    // range maximum and sum of exponentials per head
#pragma unroll
    for (int r = 0; r < NR; ++r) {
#pragma unroll
      for (int o = 16; o >= 8; o >>= 1) mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], o));
      if ((tid & 31) == 0) red[0][r][tid >> 5] = mx[r];
    }
    __syncthreads();   // scores of this range visible to the block
    float sum[NR];
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      mx[r] = fmaxf(fmaxf(red[0][r][0], red[0][r][1]), fmaxf(red[0][r][2], red[0][r][3]));
      sum[r] = 0.0f;
      for (int idx = i0 + tid; idx < i1; idx += kThreads) sum[r] += expf(sc[(int64_t)(h0 + r) * stride + idx] - mx[r]);
      sum[r] = warp_sum(sum[r]);
      if ((tid & 31) == 0) red[1][r][tid >> 5] = sum[r];
    }
    __syncthreads();
    if (tid < NR) stats[h0 + tid] = make_float2(fmaxf(fmaxf(red[0][tid][0], red[0][tid][1]), fmaxf(red[0][tid][2], red[0][tid][3])),
                                                red[1][tid][0] + red[1][tid][1] + red[1][tid][2] + red[1][tid][3]);
    __syncthreads();
  }
}

// grid (ranges, kv heads, rows): partial sums of this group's heads over one key range
template <class T, int NR>
__global__ void __launch_bounds__(kThreads) mix_values_kernel(const MixAttnArgs a, const Rows rows, int row0, int splits, int stride) {
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, H = a.heads;
  const int split = blockIdx.x, g = blockIdx.y, row = row0 + blockIdx.z;
  const int n_rep = H / a.kv_heads, DV = a.vdim_pad;
  float* mxs = sm;                          // [H] maximum
  float* inv = mxs + H;                     // [H] 1 / sum
  float* talk = inv + H;                    // [n_rep][H]
  float* p = talk + n_rep * H;              // [H][kTileKeys]
  float* w = p + H * kTileKeys;             // [n_rep][kTileKeys]
  float* red = w + n_rep * kTileKeys;       // [slots][8 * vchunks]
  const Span sp = span_of(row_pos(rows, row), a.window, a.keep_first);
  const int L = (sp.n + splits - 1) / splits, i0 = min(sp.n, split * L), i1 = min(sp.n, i0 + L);
  const float2* stats = reinterpret_cast<const float2*>(a.stats) + (int64_t)blockIdx.z * splits * H;
  for (int h = tid; h < H; h += kThreads) {
    float M = -INFINITY, S = 0.0f;
    for (int s = 0; s < splits; ++s) M = fmaxf(M, stats[s * H + h].x);
    for (int s = 0; s < splits; ++s) {
      const float2 t = stats[s * H + h];
      if (t.x > -INFINITY) S += t.y * expf(t.x - M);
    }
    mxs[h] = M;
    inv[h] = 1.0f / S;
  }
  for (int i = tid; i < n_rep * H; i += kThreads)
    talk[i] = a.talk ? a.talk[(g * n_rep) * H + i] : (i / H + g * n_rep == i % H ? 1.0f : 0.0f);
  __syncthreads();

  const float* sc = a.scores + (int64_t)blockIdx.z * H * stride;
  const T* vbase = static_cast<const T*>(a.v) + ((int64_t)row_seq(rows, row) * a.kv_heads + g) * a.capacity * DV;
  const int vchunks = DV / 8, slots = vchunks < kThreads ? kThreads / vchunks : 1;
  const int slot = tid / vchunks;
  float* out = a.part + (((int64_t)blockIdx.z * splits + split) * H + g * n_rep) * a.vdim;

  for (int c0 = 0; c0 < vchunks; c0 += kThreads) {   // value sizes above 8 * kThreads take several passes
    const int chunk = c0 + (vchunks < kThreads ? tid % vchunks : tid);
    for (int h0 = 0; h0 < n_rep; h0 += NR) {
      float acc[NR][8] = {};
      for (int t0 = i0; t0 < i1; t0 += kTileKeys) {
        const int nt = min(kTileKeys, i1 - t0);
        for (int i = tid; i < H * kTileKeys; i += kThreads) {
          const int h = i / kTileKeys, k = i % kTileKeys;
          p[i] = k < nt ? expf(sc[(int64_t)h * stride + t0 + k] - mxs[h]) * inv[h] : 0.0f;
        }
        __syncthreads();
        for (int i = tid; i < NR * kTileKeys; i += kThreads) {
          const int r = i / kTileKeys, k = i % kTileKeys;
          float s = 0.0f;
          for (int h = 0; h < H; ++h) s = fmaf(talk[(h0 + r) * H + h], p[h * kTileKeys + k], s);
          w[i] = s;
        }
        __syncthreads();
        if (slot < slots && chunk < vchunks)
          for (int k = slot; k < nt; k += slots) {
            float vf[8];
            load8(vbase + (int64_t)sp.key(t0 + k) * DV + 8 * chunk, vf);
#pragma unroll
            for (int r = 0; r < NR; ++r)
#pragma unroll
              for (int e = 0; e < 8; ++e) acc[r][e] = fmaf(w[r * kTileKeys + k], vf[e], acc[r][e]);
          }
        __syncthreads();
      }
      // add the slots
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        if (slot < slots && chunk < vchunks)
#pragma unroll
          for (int e = 0; e < 8; ++e) red[slot * 8 * min(vchunks, kThreads) + (chunk - c0) * 8 + e] = acc[r][e];
        __syncthreads();
        for (int d = tid; d < 8 * min(vchunks - c0, kThreads); d += kThreads) {
          float s = 0.0f;
          for (int k = 0; k < slots; ++k) s += red[k * 8 * min(vchunks, kThreads) + d];
          if (8 * c0 + d < a.vdim) out[(int64_t)(h0 + r) * a.vdim + 8 * c0 + d] = s;
        }
        __syncthreads();
      }
    }
  }
}

template <class TO>
__global__ void mix_reduce_kernel(const float* __restrict__ part, int splits, int n, TO* __restrict__ out, int64_t ldo, int row0) {
  const int i = blockIdx.x * kThreads + threadIdx.x;
  if (i >= n) return;
  const float* p = part + (int64_t)blockIdx.y * splits * n + i;
  float s = 0.0f;
  for (int k = 0; k < splits; ++k) s += p[(int64_t)k * n];
  out[(int64_t)(row0 + blockIdx.y) * ldo + i] = to<TO>(s);
}

int scores_stride(const MixAttnArgs& a) { return (a.max_visible + 3) & ~3; }

size_t values_smem(const MixAttnArgs& a) {
  const int n_rep = a.heads / a.kv_heads, vchunks = a.vdim_pad / 8;
  const size_t red = 8 * (size_t)(vchunks < kThreads ? (kThreads / vchunks) * vchunks : kThreads);
  return 4 * (2 * (size_t)a.heads + (size_t)n_rep * a.heads + (size_t)a.heads * kTileKeys + (size_t)n_rep * kTileKeys + red);
}

template <class T, int NR>
cudaError_t launch_rows_nr(const MixAttnArgs& a, const Rows& rows, int row0, int n, int splits, cudaStream_t st) {
  const int stride = scores_stride(a);
  const size_t s1 = 4 * (size_t)(a.heads / a.kv_heads) * a.dim_pad, s2 = values_smem(a);
  if (s1 > 200 * 1024 || s2 > 200 * 1024) return cudaErrorInvalidValue;
  cudaError_t e = cudaSuccess;
  if (s1 > 48 * 1024) e = cudaFuncSetAttribute(mix_scores_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
  if (e == cudaSuccess && s2 > 48 * 1024) e = cudaFuncSetAttribute(mix_values_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2);
  if (e != cudaSuccess) return e;
  const dim3 grid(splits, a.kv_heads, n);
  mix_scores_kernel<T, NR><<<grid, kThreads, s1, st>>>(a, rows, row0, splits, stride);
  mix_values_kernel<T, NR><<<grid, kThreads, s2, st>>>(a, rows, row0, splits, stride);
  return cudaGetLastError();
}

}  // namespace

int mix_attn_splits(const MixAttnArgs& a, int sm_count) {
  // about 32 keys per range at least, two blocks per SM at most
  int s = (a.max_visible + 31) / 32;
  const int fill = (2 * sm_count + a.kv_heads - 1) / a.kv_heads;
  if (s > fill) s = fill;
  if (s > kMixAttnMaxSplits) s = kMixAttnMaxSplits;
  return s < 1 ? 1 : s;
}

template <class T, class TO>
cudaError_t launch_mix_attention_rows(const MixAttnArgs& a, const Rows& rows, TO* out, int64_t ldo, int sm_count, cudaStream_t st, int* launches) {
  const int splits = rows.n > 64 ? 1 : mix_attn_splits(a, sm_count);
  const int n_rep = a.heads / a.kv_heads, hv = a.heads * a.vdim;
  // rows per launch: what the scratch holds
  const uint64_t per_scores = (uint64_t)a.heads * scores_stride(a), per_stats = 2ull * splits * a.heads, per_part = (uint64_t)splits * hv;
  uint64_t fit = a.scores_floats / per_scores;
  if (a.stats_floats / per_stats < fit) fit = a.stats_floats / per_stats;
  if (a.part_floats / per_part < fit) fit = a.part_floats / per_part;
  if (fit > 32768) fit = 32768;
  if (fit < 1) return cudaErrorInvalidValue;
  for (int r0 = 0; r0 < rows.n; r0 += (int)fit) {
    const int n = rows.n - r0 < (int)fit ? rows.n - r0 : (int)fit;
    cudaError_t e;
    if (n_rep % 8 == 0) e = launch_rows_nr<T, 8>(a, rows, r0, n, splits, st);
    else if (n_rep % 4 == 0) e = launch_rows_nr<T, 4>(a, rows, r0, n, splits, st);
    else if (n_rep % 3 == 0) e = launch_rows_nr<T, 3>(a, rows, r0, n, splits, st);
    else if (n_rep % 2 == 0) e = launch_rows_nr<T, 2>(a, rows, r0, n, splits, st);
    else e = launch_rows_nr<T, 1>(a, rows, r0, n, splits, st);
    if (e != cudaSuccess) return e;
    mix_reduce_kernel<TO><<<dim3((hv + kThreads - 1) / kThreads, n), kThreads, 0, st>>>(a.part, splits, hv, out, ldo, r0);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    *launches += 3;
  }
  return cudaSuccess;
}
template cudaError_t launch_mix_attention_rows<float, float>(const MixAttnArgs&, const Rows&, float*, int64_t, int, cudaStream_t, int*);
template cudaError_t launch_mix_attention_rows<__nv_bfloat16, float>(const MixAttnArgs&, const Rows&, float*, int64_t, int, cudaStream_t, int*);
template cudaError_t launch_mix_attention_rows<__nv_bfloat16, __nv_bfloat16>(const MixAttnArgs&, const Rows&, __nv_bfloat16*, int64_t, int,
                                                                             cudaStream_t, int*);

// ---- prompts on the tensor cores (mma.sync bf16).  A strip of consecutive query rows at a time, so that the scores of
// every head stay in the L2 cache between three launches:
//   scores   q . k * scale of 64 rows x 64 key columns of one head, and the {max, sum of exponentials} of each row's
//            visible columns in the tile
//   mix      per row: softmax of every head over its visible columns, then talk x weights on the tensor cores, both
//            fed as two bf16 parts (high, remainder); each mixed weight is left in two such parts in the place of its
//            score, invisible columns as zero
//   values   weights x value rows, both parts
// Column c of a strip is key c for c < kk (kept tokens below the strip's first window), else key lo + c - kk.
namespace {

constexpr int kQT = 64, kCT = 64, kMmaThreads = 128;

struct Strip {
  int row0, rows;      // rows of the batch
  int pos0;            // position of row0
  int lo, kk, cols;    // key columns; cols_pad: columns rounded up to whole tiles
  int cols_pad;
};

__device__ __forceinline__ int strip_key(const Strip& s, int c) { return c < s.kk ? c : s.lo + c - s.kk; }

// whether any of the strip's rows [i0, i0 + 64) sees a column of [c0, c0 + 64)
__device__ __forceinline__ bool tile_visible(const Strip& s, int i0, int c0, int window, int keep) {
  const int p0 = s.pos0 + i0, p1 = s.pos0 + min(i0 + kQT, s.rows) - 1;
  const int c1 = min(c0 + kCT, s.cols) - 1;
  if (c1 < c0) return false;
  const int k0 = strip_key(s, c0), k1 = strip_key(s, c1);
  if (k0 > p1) return false;
  return k0 < keep || window <= 0 || p0 - k1 < window;
}

// the visible columns of a strip's row i: [0, kept) and [w0, w1]
struct RowSpan {
  int kept, w0, w1;
  __device__ __forceinline__ bool sees(int c) const { return c < kept || (c >= w0 && c <= w1); }
};
__device__ __forceinline__ RowSpan row_span(const Strip& s, int i, int window, int keep) {
  const int pos = s.pos0 + i, lo = window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0;
  return RowSpan{min(keep, lo), s.kk + lo - s.lo, s.kk + pos - s.lo};
}

__global__ void __launch_bounds__(kMmaThreads) mix_prompt_scores_kernel(const MixAttnArgs a, const int seq, const Strip s) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int D = a.dim_pad, row_halves = D + 8;
  __nv_bfloat16* qt = reinterpret_cast<__nv_bfloat16*>(raw);      // [64][D + 8]
  __nv_bfloat16* kt = qt + kQT * row_halves;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int c0 = blockIdx.x * kCT, i0 = blockIdx.y * kQT, h = blockIdx.z, kh = h / (a.heads / a.kv_heads);
  if (!tile_visible(s, i0, c0, a.window, a.keep_first)) return;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q);
  const __nv_bfloat16* k = static_cast<const __nv_bfloat16*>(a.k) + ((int64_t)seq * a.kv_heads + kh) * a.capacity * D;
  // two threads per row
  for (int c = (tid & 1) * 8; c < D; c += 16) {
    const int r = tid >> 1;
    const bool kl = c0 + r < s.cols, ql = i0 + r < s.rows;
    cp16_zfill(kt + r * row_halves + c, k + (kl ? (int64_t)strip_key(s, c0 + r) * D + c : 0), kl);
    cp16_zfill(qt + r * row_halves + c, q + (ql ? ((int64_t)(s.row0 + i0 + r) * a.heads + h) * D + c : 0), ql);
  }
  asm volatile("cp.async.commit_group;\n" ::: "memory");
  asm volatile("cp.async.wait_group 0;\n" ::: "memory");
  __syncthreads();
  float acc[kCT / 8][4] = {};
  for (int kk = 0; kk < D / 16; ++kk) {
    uint32_t qa[4];
    ldsm(qa, qt + (16 * warp + (lane & 15)) * row_halves + 16 * kk + (lane >> 4) * 8);
#pragma unroll
    for (int nt = 0; nt < kCT / 16; ++nt) {
      uint32_t b[4];
      ldsm(b, kt + (16 * nt + (lane & 7) + (lane >> 4) * 8) * row_halves + 16 * kk + ((lane >> 3) & 1) * 8);
      mma_bf16_16816(acc[2 * nt], qa, b[0], b[1]);
      mma_bf16_16816(acc[2 * nt + 1], qa, b[2], b[3]);
    }
  }
  // the scores leave through shared memory, whole rows of the tile at a time
  constexpr int kTileRow = kCT + 4;
  float* tile = reinterpret_cast<float*>(raw);
  __syncthreads();
  // every row of the tile sees every column: the last row's window starts at or before it, the first row's ends after it
  const bool inside = row_span(s, min(i0 + kQT, s.rows) - 1, a.window, a.keep_first).w0 <= c0 && row_span(s, i0, a.window, a.keep_first).w1 >= c0 + kCT - 1;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int i = i0 + 16 * warp + g + 8 * half;
    const RowSpan span = row_span(s, i, a.window, a.keep_first);
    float m = -INFINITY, sum = 0.0f;
#pragma unroll
    for (int nt = 0; nt < kCT / 8; ++nt) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float& v = acc[nt][2 * half + e];
        v *= a.scale;
      }
      *reinterpret_cast<float2*>(tile + (16 * warp + g + 8 * half) * kTileRow + 8 * nt + 2 * t) = make_float2(acc[nt][2 * half], acc[nt][2 * half + 1]);
      if (!inside) {
#pragma unroll
        for (int e = 0; e < 2; ++e)
          if (!span.sees(c0 + 8 * nt + 2 * t + e)) acc[nt][2 * half + e] = -INFINITY;
      }
      m = fmaxf(m, fmaxf(acc[nt][2 * half], acc[nt][2 * half + 1]));
    }
    m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));   // the four lanes of a row
    m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
    const float base = m == -INFINITY ? 0.0f : m;
#pragma unroll
    for (int nt = 0; nt < kCT / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) sum += __expf(acc[nt][2 * half + e] - base);
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    if (t == 0 && i < s.rows) reinterpret_cast<float2*>(a.stats)[((int64_t)i * a.heads + h) * (s.cols_pad / kCT) + blockIdx.x] = make_float2(m, sum);
  }
  __syncwarp();   // a warp stores the 16 rows it wrote
#pragma unroll
  for (int x = lane; x < 16 * (kCT / 4); x += 32) {
    const int r = 16 * warp + x / (kCT / 4), c = x % (kCT / 4) * 4;
    if (i0 + r < s.rows)
      *reinterpret_cast<float4*>(a.scores + ((int64_t)(i0 + r) * a.heads + h) * s.cols_pad + c0 + c) = *reinterpret_cast<const float4*>(tile + r * kTileRow + c);
  }
}

constexpr int kMixThreads = 256;

// grid (rows, shares of the column tiles); heads padded to HM, a multiple of 16
template <int HM>
struct WeightsSmem {
  static constexpr int kTalkRow = HM + 8, kTileRow = kCT + 4, kStages = 3;
  float tile[kStages][HM][kTileRow];            // 64 columns of every head's scores, then of the mixed weights
  __nv_bfloat16 talk_hi[HM][kTalkRow], talk_lo[HM][kTalkRow];
  float mx[HM], inv[HM];
};
template <int HM>
__global__ void __launch_bounds__(kMixThreads) mix_prompt_weights_kernel(const MixAttnArgs a, const Strip s) {
  constexpr int MT = HM / 16;
  static_assert(kMixThreads / 32 * 8 == kCT, "eight columns per warp");
  extern __shared__ __align__(16) unsigned char raw[];
  WeightsSmem<HM>& sm = *reinterpret_cast<WeightsSmem<HM>*>(raw);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3, H = a.heads;
  const int i = blockIdx.x, tiles = s.cols_pad / kCT, q_tile = i / kQT * kQT;
  const RowSpan span = row_span(s, i, a.window, a.keep_first);
  float* sc = a.scores + (int64_t)i * H * s.cols_pad;
  auto next = [&](int b) {
    while (b < tiles && !tile_visible(s, q_tile, b * kCT, a.window, a.keep_first)) b += gridDim.y;
    return b;
  };
  auto issue = [&](int b, int buf) {
    if (b < tiles)
      for (int x = tid; x < H * (kCT / 4); x += kMixThreads) {
        const int h = x / (kCT / 4), c = x % (kCT / 4) * 4;
        cp16_zfill(&sm.tile[buf][h][c], sc + (int64_t)h * s.cols_pad + b * kCT + c, true);
      }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  int b0 = next(blockIdx.y), b1 = next(b0 + gridDim.y), buf = 0;
  issue(b0, 0);
  issue(b1, 1);
  for (int x = tid; x < HM * HM; x += kMixThreads) {
    const int h = x / HM, k = x % HM;
    const float v = h < H && k < H ? (a.talk ? a.talk[h * H + k] : (h == k ? 1.0f : 0.0f)) : 0.0f;
    const __nv_bfloat16 hi = __float2bfloat16_rn(v);
    sm.talk_hi[h][k] = hi;
    sm.talk_lo[h][k] = __float2bfloat16_rn(v - __bfloat162float(hi));
  }
  for (int h = warp; h < HM; h += kMixThreads / 32) {
    const float2* st = reinterpret_cast<const float2*>(a.stats) + ((int64_t)i * H + h) * tiles;
    float m = -INFINITY, sum = 0.0f;
    for (int b = lane; h < H && b < tiles; b += 32)
      if (tile_visible(s, q_tile, b * kCT, a.window, a.keep_first)) {
        const float2 v = st[b];
        const float to = fmaxf(m, v.x);
        if (to > -INFINITY) sum = sum * __expf(m - to) + v.y * __expf(v.x - to);
        m = to;
      }
    float M = m;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    sum = warp_sum(m > -INFINITY ? sum * __expf(m - M) : 0.0f);
    if (lane == 0) {
      sm.mx[h] = h < H ? M : 0.0f;
      sm.inv[h] = h < H ? 1.0f / sum : 0.0f;
    }
  }
  __syncthreads();
  // 8 columns per warp: weights of all heads as the B operand (k = head, n = column), mixed ones as C
  while (b0 < tiles) {
    asm volatile("cp.async.wait_group 1;\n" ::: "memory");
    __syncthreads();   // this tile has landed; the one before it has been stored
    const int b2 = next(b1 + gridDim.y);
    issue(b2, buf == 0 ? 2 : buf - 1);
    float (*tile)[WeightsSmem<HM>::kTileRow] = sm.tile[buf];
    const int c0 = 8 * warp;
    const bool sees = span.sees(b0 * kCT + c0 + g);
    uint32_t hi[MT][2], lo[MT][2];
#pragma unroll
    for (int kt = 0; kt < MT; ++kt) {
      float p[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = 16 * kt + 2 * t + (e & 1) + 8 * (e >> 1);
        p[e] = sees && h < H ? __expf(tile[h][c0 + g] - sm.mx[h]) * sm.inv[h] : 0.0f;
      }
      split2(p[0], p[1], hi[kt][0], lo[kt][0]);
      split2(p[2], p[3], hi[kt][1], lo[kt][1]);
    }
    __syncwarp();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      float w[4] = {};
#pragma unroll
      for (int kt = 0; kt < MT; ++kt) {
        uint32_t th[4], tl[4];
        ldsm(th, &sm.talk_hi[16 * mt + (lane & 15)][16 * kt + (lane >> 4) * 8]);
        ldsm(tl, &sm.talk_lo[16 * mt + (lane & 15)][16 * kt + (lane >> 4) * 8]);
        mma_bf16_16816(w, th, hi[kt][0], hi[kt][1]);
        mma_bf16_16816(w, th, lo[kt][0], lo[kt][1]);
        mma_bf16_16816(w, tl, hi[kt][0], hi[kt][1]);
      }
      // every lane's scores of the warp's columns are in its operands by now: their places are free
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int h = 16 * mt + g + 8 * half;
        if (h >= H) continue;
        uint32_t wh, wl;
        split2(w[2 * half], w[2 * half + 1], wh, wl);
        *reinterpret_cast<uint2*>(&tile[h][c0 + 2 * t]) = make_uint2(__byte_perm(wh, wl, 0x5410), __byte_perm(wh, wl, 0x7632));
      }
    }
    __syncthreads();
    for (int x = tid; x < H * (kCT / 4); x += kMixThreads) {
      const int h = x / (kCT / 4), c = x % (kCT / 4) * 4;
      *reinterpret_cast<float4*>(sc + (int64_t)h * s.cols_pad + b0 * kCT + c) = *reinterpret_cast<const float4*>(&tile[h][c]);
    }
    b0 = b1;
    b1 = b2;
    buf = buf == 2 ? 0 : buf + 1;
  }
}

template <int HM>
cudaError_t launch_prompt_weights(const MixAttnArgs& a, const Strip& s, cudaStream_t st) {
  const int smem = (int)sizeof(WeightsSmem<HM>), tiles = s.cols_pad / kCT;
  const cudaError_t e = cudaFuncSetAttribute(mix_prompt_weights_kernel<HM>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  mix_prompt_weights_kernel<HM><<<dim3(s.rows, tiles > 12 ? 3 : tiles > 6 ? 2 : 1), kMixThreads, smem, st>>>(a, s);
  return cudaGetLastError();
}

// grid (query tiles, heads, blocks of 8 NT value columns).  Eight warps: 16 query rows each, twice -- the second four
// warps take the second half of every key tile, and the halves are added at the end
constexpr int kValuesThreads = 256, kValuesStages = 3;
template <int NT>
struct ValuesSmem {
  static constexpr int kWRow = kCT + 4, kVRow = 8 * NT + 8;
  uint32_t w[kValuesStages][kQT][kWRow];
  __nv_bfloat16 v[kValuesStages][kCT][kVRow];
};
template <int NT>
__global__ void __launch_bounds__(kValuesThreads) mix_prompt_values_kernel(const MixAttnArgs a, const int seq, const Strip s, __nv_bfloat16* __restrict__ out,
                                                                        int64_t ldo) {
  extern __shared__ __align__(16) unsigned char raw[];
  ValuesSmem<NT>& sm = *reinterpret_cast<ValuesSmem<NT>*>(raw);
  const int tid = threadIdx.x, lane = tid & 31, warp = (tid >> 5) & 3, half_of_keys = tid >> 7, g = lane >> 2, t = lane & 3;
  const int i0 = blockIdx.x * kQT, h = blockIdx.y, v0 = blockIdx.z * 8 * NT, n_rep = a.heads / a.kv_heads;
  const uint32_t* w = reinterpret_cast<const uint32_t*>(a.scores);
  const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(a.v) + ((int64_t)seq * a.kv_heads + h / n_rep) * a.capacity * a.vdim_pad;
  auto issue = [&](int c0, int buf) {
    for (int i = tid; i < kQT * (kCT / 4); i += kValuesThreads) {
      const int r = i / (kCT / 4), c = i % (kCT / 4) * 4;
      const bool live = i0 + r < s.rows;
      cp16_zfill(&sm.w[buf][r][c], w + (live ? ((int64_t)(i0 + r) * a.heads + h) * s.cols_pad + c0 + c : 0), live);
    }
    for (int i = tid; i < kCT * NT; i += kValuesThreads) {
      const int r = i / NT, c = i % NT * 8;
      const bool live = c0 + r < s.cols && v0 + c < a.vdim_pad;
      cp16_zfill(&sm.v[buf][r][c], v + (live ? (int64_t)strip_key(s, c0 + r) * a.vdim_pad + v0 + c : 0), live);
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  auto next = [&](int c0) {
    while (c0 < s.cols_pad && !tile_visible(s, i0, c0, a.window, a.keep_first)) c0 += kCT;
    return c0;
  };
  float acc[NT][4] = {};
  // a ring of three tiles, two of them on their way while one is worked on
  int ahead = next(0), work = 0, fill = 0, pending = 0;
  auto feed = [&]() {
    if (ahead < s.cols_pad) {
      issue(ahead, fill);
      fill = fill == kValuesStages - 1 ? 0 : fill + 1;
      ahead = next(ahead + kCT);
      ++pending;
    } else {
      asm volatile("cp.async.commit_group;\n" ::: "memory");   // empty, so that the count below holds
    }
  };
  feed();
  feed();
  for (; pending > 0; --pending) {
    asm volatile("cp.async.wait_group 1;\n" ::: "memory");
    __syncthreads();   // the tile has landed, and the one worked on before it is free
    feed();
    const int buf = work;
    work = work == kValuesStages - 1 ? 0 : work + 1;
#pragma unroll
    for (int kh = 0; kh < kCT / 32; ++kh) {
      const int kk = 2 * half_of_keys + kh;
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int part = 0; part < 4; ++part) {
        const uint2 x = *reinterpret_cast<const uint2*>(&sm.w[buf][16 * warp + g + 8 * (part & 1)][16 * kk + 2 * t + 8 * (part >> 1)]);
        hi[part] = __byte_perm(x.x, x.y, 0x5410);
        lo[part] = __byte_perm(x.x, x.y, 0x7632);
      }
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        uint32_t b[4];
        ldsm_trans(b, &sm.v[buf][16 * kk + (lane & 15)][16 * np + (lane >> 4) * 8]);
        mma_bf16_16816(acc[2 * np], hi, b[0], b[1]);
        mma_bf16_16816(acc[2 * np], lo, b[0], b[1]);
        mma_bf16_16816(acc[2 * np + 1], hi, b[2], b[3]);
        mma_bf16_16816(acc[2 * np + 1], lo, b[2], b[3]);
      }
    }
  }
  __syncthreads();
  // add the halves through shared memory 
  float* sum = reinterpret_cast<float*>(raw) + (tid & 127);
  static_assert(sizeof(ValuesSmem<NT>) >= 4 * 128 * 4 * NT, "room for one half's accumulators");
  if (half_of_keys == 1)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) sum[128 * (4 * nt + e)] = acc[nt][e];
  __syncthreads();
  if (half_of_keys == 1) return;
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[nt][e] += sum[128 * (4 * nt + e)];
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int i = i0 + 16 * warp + g + 8 * half;
    if (i >= s.rows) continue;
    __nv_bfloat16* o = out + (int64_t)(s.row0 + i) * ldo + h * a.vdim;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = v0 + 8 * nt + 2 * t + e;
        if (c < a.vdim) o[c] = __float2bfloat16_rn(acc[nt][2 * half + e]);
      }
  }
}

template <int NT>
cudaError_t launch_prompt_values(const MixAttnArgs& a, int seq, const Strip& s, __nv_bfloat16* out, int64_t ldo, cudaStream_t st) {
  const int smem = (int)sizeof(ValuesSmem<NT>);
  const cudaError_t e = cudaFuncSetAttribute(mix_prompt_values_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  mix_prompt_values_kernel<NT><<<dim3((s.rows + kQT - 1) / kQT, a.heads, (a.vdim_pad + 8 * NT - 1) / (8 * NT)), kValuesThreads, smem, st>>>(a, seq, s, out, ldo);
  return cudaGetLastError();
}

// key columns of the strip of `rows` query rows from position pos0
Strip make_strip(const MixAttnArgs& a, int row0, int rows, int pos0) {
  Strip s{};
  s.row0 = row0;
  s.rows = rows;
  s.pos0 = pos0;
  s.lo = a.window > 0 && pos0 - a.window + 1 > 0 ? pos0 - a.window + 1 : 0;
  s.kk = a.keep_first < s.lo ? a.keep_first : s.lo;
  s.cols = s.kk + pos0 + rows - s.lo;
  s.cols_pad = (s.cols + kCT - 1) / kCT * kCT;
  return s;
}

}  // namespace

bool mix_attention_prompt_supported(const MixAttnArgs& a) {
  // one tile of query rows must fit the scratch
  const uint64_t widest = ((uint64_t)a.max_visible + 2 * kQT + kCT) * a.heads * kQT;
  return a.heads <= 64 && a.dim_pad % 16 == 0 && a.dim_pad <= 256 && widest <= a.scores_floats && widest / 32 <= a.stats_floats;
}

cudaError_t launch_mix_attention_prompt(const MixAttnArgs& a, const Rows& rows, int pos0, __nv_bfloat16* out, int64_t ldo, cudaStream_t st,
                                        int* launches) {
  int smem = 2 * kQT * (a.dim_pad + 8) * 2;
  if (smem < kQT * (kCT + 4) * 4) smem = kQT * (kCT + 4) * 4;
  cudaError_t e = cudaSuccess;
  if (smem > 48 * 1024) e = cudaFuncSetAttribute(mix_prompt_scores_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  for (int r0 = 0; e == cudaSuccess && r0 < rows.n;) {
    // as many 64-row tiles as the scratch holds, at most 256 rows (a longer strip adds columns few of its rows see)
    int n = rows.n - r0 < kQT ? rows.n - r0 : kQT;
    Strip s = make_strip(a, r0, n, pos0 + r0);
    while (n < rows.n - r0 && n < 256) {
      const int more = rows.n - r0 < n + kQT ? rows.n - r0 : n + kQT;
      const Strip t = make_strip(a, r0, more, pos0 + r0);
      if ((uint64_t)t.rows * a.heads * t.cols_pad > a.scores_floats || (uint64_t)t.rows * a.heads * t.cols_pad / 32 > a.stats_floats) break;
      n = more;
      s = t;
    }
    mix_prompt_scores_kernel<<<dim3(s.cols_pad / kCT, (n + kQT - 1) / kQT, a.heads), kMmaThreads, smem, st>>>(a, rows.seq0, s);
    e = cudaGetLastError();
    if (e != cudaSuccess) break;
    e = a.heads <= 16 ? launch_prompt_weights<16>(a, s, st) : a.heads <= 32 ? launch_prompt_weights<32>(a, s, st) : launch_prompt_weights<64>(a, s, st);
    if (e != cudaSuccess) break;
    if (a.vdim_pad <= 32) e = launch_prompt_values<4>(a, rows.seq0, s, out, ldo, st);
    else e = launch_prompt_values<8>(a, rows.seq0, s, out, ldo, st);
    *launches += 3;
    r0 += n;
  }
  return e;
}

}  // namespace emelb
