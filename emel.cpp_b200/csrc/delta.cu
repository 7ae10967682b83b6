// Gated delta rule: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q / sqrt(dim), one decay g and one step size
// beta per head and token, q and k unit vectors behind a short causal convolution and silu.  The state [dim][vdim] of a
// (sequence, head) is f32 and stays in HBM between calls; a sequence that starts at position 0 starts from zero whatever
// the memory holds.
//
// One token: everything from the projections to the gated heads is one launch, a cluster per (head, row).
// Prompts: convolution and the tokens' scalars; the recurrence; norm and gate.  1 / |q| and 1 / |k| stay f32 factors
// beside the convolved vectors, so that the vectors themselves can be bf16 operands.
#include <cooperative_groups.h>
#include <math.h>

#include "act.cuh"
#include "common.cuh"
#include "layered.h"
#include "mma_bf16.cuh"

namespace emelb {
namespace {

__device__ __forceinline__ float from(float x) { return x; }
__device__ __forceinline__ float from(__nv_bfloat16 x) { return __bfloat162float(x); }
template <class T> __device__ __forceinline__ T to(float x);
template <> __device__ __forceinline__ float to<float>(float x) { return x; }
template <> __device__ __forceinline__ __nv_bfloat16 to<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }

constexpr float kUnitEps = 1e-6f;   // inside the root of the unit norms

__device__ __forceinline__ float log_decay(const DeltaArgs& a, int h, float x) { return -expf(a.decay_log[h]) * softplusf_(x + a.step_bias[h]); }

// ---- one token.  The channels of one head's q, k (and `nv` of its values from v0) through convolution and silu into shared
// memory: q [dim] | k [dim] | v; the ring takes the step's projections (keys and queries once per group of heads).
template <class TP>
__device__ __forceinline__ void step_inputs(const DeltaArgs& a, const TP* x, float* ring, int pos, int h, int v0, int nv, bool store_qk, float* dst) {
  const int rep = a.heads / a.kv_heads, kh = h / rep, channels = a.channels();
  for (int i = threadIdx.x; i < 2 * a.dim + nv; i += blockDim.x) {
    const int c = i < a.dim ? kh * a.dim + i : i < 2 * a.dim ? (a.kv_heads + kh) * a.dim + i - a.dim : 2 * a.kv_heads * a.dim + h * a.vdim + v0 + i - 2 * a.dim;
    const float u = from(x[c]);
    float y = a.conv[(int64_t)(a.taps - 1) * channels + c] * u;
#pragma unroll 4
    for (int b = 1; b < a.taps; ++b) {
      const float past = b <= pos ? ring[(int64_t)((pos - b) % a.taps) * channels + c] : 0.0f;
      y = fmaf(a.conv[(int64_t)(a.taps - 1 - b) * channels + c], past, y);
    }
    // no block reads this entry in this step: its old token lies `taps` back
    if (i >= 2 * a.dim || (store_qk && h % rep == 0)) ring[(int64_t)(pos % a.taps) * channels + c] = u;
    dst[i] = siluf_(y);
  }
}
// after a barrier, by the first three warps: 1 / |q| / sqrt(dim), 1 / |k|, q . k (unscaled)
__device__ __forceinline__ void step_scalars(const DeltaArgs& a, const float* q, const float* k, float* scal) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp >= 3) return;
  const float *s0 = warp == 1 ? k : q, *s1 = warp == 0 ? q : k;
  float s = 0.0f;
  for (int i = lane; i < a.dim; i += 32) s = fmaf(s0[i], s1[i], s);
  s = warp_sum(s);
  if (lane == 0) scal[warp] = warp == 2 ? s : 1.0f / sqrtf(s + kUnitEps) * (warp == 0 ? 1.0f / sqrtf((float)a.dim) : 1.0f);
}

// A cluster = one head of one row, a block = 32 of its value columns; the state tile stays in registers between its two
// uses, and the blocks add their squares through distributed shared memory.  Grid (column tiles, heads, rows).
constexpr int kTileCols = 32, kTileGroups = 16, kTileThreads = kTileCols * kTileGroups, kTileRows = 8;   // dim <= 128
constexpr int kMaxTiles = 8;

template <class TP, class TO>
__global__ void __launch_bounds__(kTileThreads) delta_step_kernel(const DeltaArgs a, const Rows rows, TO* __restrict__ out, int64_t ldo) {
  namespace cg = cooperative_groups;
  extern __shared__ float sm[];
  float *q = sm, *k = q + a.dim, *v = k + a.dim;           // [dim], [dim], [kTileCols]
  __shared__ float red[2][kTileGroups][kTileCols];
  __shared__ float scal[3], squares;
  pdl_trigger();
  pdl_wait();
  cg::cluster_group cluster = cg::this_cluster();
  const int v0 = blockIdx.x * kTileCols, h = blockIdx.y, r = blockIdx.z, cols = threadIdx.x % kTileCols, group = threadIdx.x / kTileCols;
  const int pos = rows.prompt ? rows.pos[0] : rows.pos[r], seq = rows.prompt ? rows.seq0 : rows.seq0 + r, c = v0 + cols;
  const bool live = c < a.vdim;
  float* state = a.state + ((int64_t)seq * a.heads + h) * a.dim * a.vdim;
  float S[kTileRows];
#pragma unroll
  for (int i = 0; i < kTileRows; ++i) {
    const int row = group + i * kTileGroups;
    S[i] = pos > 0 && row < a.dim && live ? state[(int64_t)row * a.vdim + c] : 0.0f;
  }
  const float* gates = a.gates + (int64_t)r * a.ldg;
  const float step = gates[h], decay = gates[a.heads + h];
  const TP* x = static_cast<const TP*>(a.proj) + (int64_t)r * a.ldp;
  const float gate = live ? from(x[a.channels() + h * a.vdim + c]) : 0.0f;
  step_inputs(a, x, a.conv_state + (int64_t)seq * a.taps * a.channels(), pos, h, v0, min(kTileCols, a.vdim - v0), blockIdx.x == 0, sm);
  __syncthreads();
  step_scalars(a, q, k, scal);
  float sk = 0.0f, sq = 0.0f;
#pragma unroll
  for (int i = 0; i < kTileRows; ++i) {
    const int row = group + i * kTileGroups;
    if (row < a.dim) {
      sk = fmaf(S[i], k[row], sk);
      sq = fmaf(S[i], q[row], sq);
    }
  }
  red[0][group][cols] = sk;
  red[1][group][cols] = sq;
  __syncthreads();
  sk = sq = 0.0f;
#pragma unroll
  for (int i = 0; i < kTileGroups; ++i) {
    sk += red[0][i][cols];
    sq += red[1][i][cols];
  }
  const float beta = sigmoidf_(step), g = expf(log_decay(a, h, decay)), rq = scal[0], rk = scal[1];
  const float u = live ? beta * (v[cols] - g * rk * sk) : 0.0f, o = live ? g * rq * sq + scal[2] * rq * rk * u : 0.0f;
  if (live) {
#pragma unroll
    for (int i = 0; i < kTileRows; ++i) {
      const int row = group + i * kTileGroups;
      if (row < a.dim) state[(int64_t)row * a.vdim + c] = fmaf(k[row], rk * u, g * S[i]);
    }
  }
  if (group == 0) {
    const float ss = warp_sum(o * o);
    if (cols == 0) squares = ss;
  }
  cluster.sync();
  if (group == 0) {
    const float mine = cols < (int)gridDim.x ? *cluster.map_shared_rank(&squares, cols) : 0.0f;
    const float inv = 1.0f / sqrtf(warp_sum(mine) / a.vdim + a.eps);
    if (live) out[(int64_t)r * ldo + h * a.vdim + c] = to<TO>(o * inv * a.norm[c] * siluf_(gate));
  }
  cluster.sync();   // no block leaves while another reads its sum
}

// other sizes: one block per (head, row), the state read twice
constexpr int kStepThreads = 512, kStepCols = 128, kStepGroups = kStepThreads / kStepCols;

template <class TP, class TO>
__global__ void __launch_bounds__(kStepThreads) delta_step_wide_kernel(const DeltaArgs a, const Rows rows, TO* __restrict__ out, int64_t ldo) {
  extern __shared__ float sm[];
  float *q = sm, *k = q + a.dim, *v = k + a.dim;          // [dim], [dim], [vdim] (later the outputs)
  float* red = v + a.vdim;                                // [2][kStepGroups][kStepCols]
  __shared__ float scal[3], total[kStepThreads / 32];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, cols = tid % kStepCols, group = tid / kStepCols;
  const int pos = rows.prompt ? rows.pos[0] : rows.pos[r], seq = rows.prompt ? rows.seq0 : rows.seq0 + r;
  float* state = a.state + ((int64_t)seq * a.heads + h) * a.dim * a.vdim;
  const TP* x = static_cast<const TP*>(a.proj) + (int64_t)r * a.ldp;
  step_inputs(a, x, a.conv_state + (int64_t)seq * a.taps * a.channels(), pos, h, 0, a.vdim, true, sm);
  __syncthreads();
  step_scalars(a, q, k, scal);
  const float* gates = a.gates + (int64_t)r * a.ldg;
  const float beta = sigmoidf_(gates[h]), g = expf(log_decay(a, h, gates[a.heads + h]));
  __syncthreads();
  const float rq = scal[0], rk = scal[1], qk = scal[2] * rq * rk;
  float ss = 0.0f;
  for (int c0 = 0; c0 < a.vdim; c0 += kStepCols) {
    const int c = c0 + cols;
    const bool live = c < a.vdim;
    float sk = 0.0f, sq = 0.0f;
    if (live && pos > 0) {
#pragma unroll 8
      for (int row = group; row < a.dim; row += kStepGroups) {
        const float s = state[(int64_t)row * a.vdim + c];
        sk = fmaf(s, k[row], sk);
        sq = fmaf(s, q[row], sq);
      }
    }
    red[group * kStepCols + cols] = sk;
    red[(kStepGroups + group) * kStepCols + cols] = sq;
    __syncthreads();
    sk = sq = 0.0f;
#pragma unroll
    for (int i = 0; i < kStepGroups; ++i) {
      sk += red[i * kStepCols + cols];
      sq += red[(kStepGroups + i) * kStepCols + cols];
    }
    const float u = live ? beta * (v[c] - g * rk * sk) : 0.0f;
    const float o = g * rq * sq + qk * u;
    __syncthreads();
    if (live) {
#pragma unroll 8
      for (int row = group; row < a.dim; row += kStepGroups) {
        const float s = pos > 0 ? state[(int64_t)row * a.vdim + c] : 0.0f;
        state[(int64_t)row * a.vdim + c] = fmaf(k[row], rk * u, g * s);
      }
      if (group == 0) {
        v[c] = o;
        ss = fmaf(o, o, ss);
      }
    }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) total[tid >> 5] = ss;
  __syncthreads();
  ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kStepCols / 32; ++i) ss += total[i];   // the first group's warps
  const float inv = 1.0f / sqrtf(ss / a.vdim + a.eps);
  const TP* gate = x + a.channels() + h * a.vdim;
  for (int c = tid; c < a.vdim; c += kStepThreads) out[(int64_t)r * ldo + h * a.vdim + c] = to<TO>(v[c] * inv * a.norm[c] * siluf_(from(gate[c])));
}

// ---- prompts
constexpr int kConvThreads = 128, kConvRows = 8;

template <class T, int V>
struct Vec;
template <class T>
struct Vec<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&f)[1]) { f[0] = from(*p); }
  static __device__ __forceinline__ void store(T* p, const float (&f)[1]) { *p = to<T>(f[0]); }
};
template <>
struct Vec<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&f)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};
template <>
struct Vec<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[4]) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack2(v.x), b = unpack2(v.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&f)[4]) {
    __nv_bfloat162 x[2] = {__floats2bfloat162_rn(f[0], f[1]), __floats2bfloat162_rn(f[2], f[3])};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(x);
  }
};

// a warp = one head's vector (query, key or value) of kConvRows consecutive rows, V channels per lane and turn; one more
// warp per block row takes the rows' gates.  Rows before the batch come from the ring.
// FEW: at most four taps, every input and weight of a turn requested at once
template <class T, int V, bool FEW>
__global__ void __launch_bounds__(kConvThreads, 5) delta_conv_kernel(const DeltaArgs a, const Rows rows) {
  const int lane = threadIdx.x & 31, task = blockIdx.x * (kConvThreads / 32) + (threadIdx.x >> 5), r0 = blockIdx.y * kConvRows;
  const int vectors = 2 * a.kv_heads + a.heads, channels = a.channels(), pos0 = rows.pos[0], nr = min(kConvRows, rows.n - r0);
  const int ns = a.scalar_count();
  if (task > vectors) return;
  if (task == vectors) {
    for (int i = lane; i < nr * a.heads; i += 32) {
      const int r = r0 + i / a.heads, h = i % a.heads;
      const float* gates = a.gates + (int64_t)r * a.ldg;
      float* s = a.scalars + (int64_t)r * ns + 2 * a.kv_heads;
      s[h] = sigmoidf_(gates[h]);
      s[a.heads + h] = log_decay(a, h, gates[a.heads + h]);
    }
    return;
  }
  const bool value = task >= 2 * a.kv_heads;
  const int size = value ? a.vdim : a.dim, base = value ? 2 * a.kv_heads * a.dim + (task - 2 * a.kv_heads) * a.vdim : task * a.dim;
  const T* proj = static_cast<const T*>(a.proj);
  T* dst = static_cast<T*>(a.qkv);
  const float* ring = a.conv_state + (int64_t)rows.seq0 * a.taps * channels;
  float ss[kConvRows] = {};
  for (int c = base + V * lane; c < base + size; c += 32 * V) {
    float y[kConvRows][V] = {};
    auto input = [&](int r, float (&u)[V]) {
      if (r >= 0 && r < rows.n) {
        Vec<T, V>::load(proj + (int64_t)r * a.ldp + c, u);
      } else if (r < 0 && pos0 + r >= 0) {
        Vec<float, V>::load(ring + (int64_t)((pos0 + r) % a.taps) * channels + c, u);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = 0.0f;
      }
    };
    if (FEW) {
      float u[kConvRows + 3][V], w[4][V];
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        if (b < a.taps) {
          Vec<float, V>::load(a.conv + (int64_t)(a.taps - 1 - b) * channels + c, w[b]);
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e) w[b][e] = 0.0f;
        }
      }
#pragma unroll
      for (int i = 0; i < kConvRows + 3; ++i) input(i >= 3 || 3 - i < a.taps ? r0 - 3 + i : rows.n, u[i]);
#pragma unroll
      for (int i = 0; i < kConvRows; ++i)
#pragma unroll
        for (int b = 3; b >= 0; --b)
#pragma unroll
          for (int e = 0; e < V; ++e) y[i][e] = fmaf(w[b][e], u[i + 3 - b][e], y[i][e]);
    } else {
      // the input of row r meets the rows r .. r + taps - 1
      for (int r = r0 - (a.taps - 1); r < r0 + nr; ++r) {
        float u[V];
        input(r, u);
#pragma unroll
        for (int i = 0; i < kConvRows; ++i) {
          const int back = r0 + i - r;
          if (back < 0 || back >= a.taps) continue;
          float w[V];
          Vec<float, V>::load(a.conv + (int64_t)(a.taps - 1 - back) * channels + c, w);
#pragma unroll
          for (int e = 0; e < V; ++e) y[i][e] = fmaf(w[e], u[e], y[i][e]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < kConvRows; ++i) {
      if (i >= nr) break;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        y[i][e] = from(to<T>(siluf_(y[i][e])));   // the norm is that of the vector as stored
        ss[i] = fmaf(y[i][e], y[i][e], ss[i]);
      }
      Vec<T, V>::store(dst + (int64_t)(r0 + i) * a.ldc + c, y[i]);
    }
  }
  if (value) return;
#pragma unroll
  for (int i = 0; i < kConvRows; ++i) {
    const float s = warp_sum(ss[i]);
    if (lane == 0 && i < nr)
      a.scalars[(int64_t)(r0 + i) * ns + task] = 1.0f / sqrtf(s + kUnitEps) * (task < a.kv_heads ? 1.0f / sqrtf((float)a.dim) : 1.0f);
  }
}

template <class T>
__global__ void delta_ring_kernel(const DeltaArgs a, const Rows rows) {
  const int c = blockIdx.x * kConvThreads + threadIdx.x, channels = a.channels(), pos0 = rows.pos[0];
  if (c >= channels) return;
  float* ring = a.conv_state + (int64_t)rows.seq0 * a.taps * channels + c;
  for (int r = max(0, rows.n - a.taps); r < rows.n; ++r) ring[(int64_t)((pos0 + r) % a.taps) * channels] = from(static_cast<const T*>(a.proj)[(int64_t)r * a.ldp + c]);
}

constexpr int kCols = 32, kGroups = 8;   // value columns per block x row groups of the state

// token by token: grid (heads, column tiles)
template <class T>
__global__ void __launch_bounds__(kCols * kGroups) delta_rows_kernel(const DeltaArgs a, const Rows rows) {
  extern __shared__ float sm[];
  float* S = sm;                              // [dim][kCols]
  float* ks = S + a.dim * kCols;              // [dim]
  float* qs = ks + a.dim;                     // [dim]
  float* red = qs + a.dim;                    // [3][kGroups][kCols]
  const int h = blockIdx.x, tx = threadIdx.x, ty = threadIdx.y, col = blockIdx.y * kCols + tx, tid = ty * kCols + tx;
  const int kh = h / (a.heads / a.kv_heads), ns = a.scalar_count();
  const bool live = col < a.vdim, carried = rows.pos[0] > 0;
  float* state = a.state + ((int64_t)rows.seq0 * a.heads + h) * a.dim * a.vdim;
  for (int i = ty; i < a.dim; i += kGroups) S[i * kCols + tx] = live && carried ? state[(int64_t)i * a.vdim + col] : 0.0f;
  for (int r = 0; r < rows.n; ++r) {
    const T* row = static_cast<const T*>(a.qkv) + (int64_t)r * a.ldc;
    const float* sc = a.scalars + (int64_t)r * ns;
    const float rq = sc[kh], rk = sc[a.kv_heads + kh], beta = sc[2 * a.kv_heads + h], g = expf(sc[2 * a.kv_heads + a.heads + h]);
    __syncthreads();
    for (int i = tid; i < a.dim; i += kCols * kGroups) {
      qs[i] = rq * from(row[kh * a.dim + i]);
      ks[i] = rk * from(row[(a.kv_heads + kh) * a.dim + i]);
    }
    const float v = live ? from(row[2 * a.kv_heads * a.dim + h * a.vdim + col]) : 0.0f;
    __syncthreads();
    float sk = 0.0f, sq = 0.0f, qk = 0.0f;
    for (int i = ty; i < a.dim; i += kGroups) {
      const float s = g * S[i * kCols + tx];
      S[i * kCols + tx] = s;
      sk = fmaf(ks[i], s, sk);
      sq = fmaf(qs[i], s, sq);
      qk = fmaf(qs[i], ks[i], qk);
    }
    red[ty * kCols + tx] = sk;
    red[(kGroups + ty) * kCols + tx] = sq;
    red[(2 * kGroups + ty) * kCols + tx] = qk;
    __syncthreads();
    sk = sq = qk = 0.0f;
#pragma unroll
    for (int i = 0; i < kGroups; ++i) {
      sk += red[i * kCols + tx];
      sq += red[(kGroups + i) * kCols + tx];
      qk += red[(2 * kGroups + i) * kCols + tx];
    }
    const float u = beta * (v - sk);
    for (int i = ty; i < a.dim; i += kGroups) S[i * kCols + tx] = fmaf(ks[i], u, S[i * kCols + tx]);
    if (ty == 0 && live) a.o[((int64_t)r * a.heads + h) * a.vdim + col] = fmaf(qk, u, sq);
  }
  if (live)
    for (int i = ty; i < a.dim; i += kGroups) state[(int64_t)i * a.vdim + col] = S[i * kCols + tx];
}

// ---- prompts on the tensor cores (mma.sync bf16, f32 accumulators), chunks of 64 tokens.  With G_i the sum of the log decays
// of a chunk's tokens up to i, S the state before the chunk, and k, q, v its rows (unit keys and scaled queries):
//   (I + A) U = R,  A_ij = beta_i exp(G_i - G_j) (k_i . k_j) for j < i,  R_i = beta_i (v_i - exp(G_i) S^T k_i)
//   o_i = exp(G_i) S^T q_i + sum_(j<=i) P_ij u_j,  P_ij = exp(G_i - G_j) (q_i . k_j)
//   S' = exp(G_n) S + sum_j exp(G_n - G_j) k_j u_j^T
// A first launch, over all chunks at once, leaves T = (I + A)^-1 (forward substitution in f32), P and the rows' factors; the
// second walks the chunks.  The convolved vectors are bf16 operands as they are, 1 / |k| and 1 / |q| are among the factors;
// every f32 matrix (T, P, R, U, the state) is fed as two bf16 operands, high part and remainder.
constexpr int kChunk = 64;
// per (chunk, head): T and P {64, 64} as packed (high, remainder) pairs, then the rows' factors
constexpr int kFactorsAt = 2 * kChunk * kChunk;
enum Factor { F_KEY = 0, F_QUERY = kChunk, F_BETA = 2 * kChunk, F_STATE = 3 * kChunk, F_LAST = 4 * kChunk, F_COUNT = 4 * kChunk + 4 };
constexpr int kChunkWords = kFactorsAt + F_COUNT;

__device__ __forceinline__ uint2 pack_pair(float x, float y) {
  uint32_t hi, lo;
  split2(x, y, hi, lo);
  return make_uint2(__byte_perm(hi, lo, 0x5410), __byte_perm(hi, lo, 0x7632));
}
// A operand rows r0 .. r0 + 15, columns c0 .. c0 + 15 of a packed matrix in shared memory
template <int LD>
__device__ __forceinline__ void load_packed(const uint32_t (*m)[LD], int r0, int c0, uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  const int lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int part = 0; part < 4; ++part) {
    const uint2 x = *reinterpret_cast<const uint2*>(&m[r0 + g + 8 * (part & 1)][c0 + 2 * t + 8 * (part >> 1)]);
    hi[part] = __byte_perm(x.x, x.y, 0x5410);
    lo[part] = __byte_perm(x.x, x.y, 0x7632);
  }
}

constexpr int kPrepThreads = 128;
template <int D>
struct PrepSmem {
  static constexpr int kRow = D + 8;
  __nv_bfloat16 q[kChunk][kRow], k[kChunk][kRow];
  float A[kChunk][kChunk + 4];
  float G[kChunk], rq[kChunk], rk[kChunk], beta[kChunk];
};

// grid (chunks, heads)
template <int D>
__global__ void __launch_bounds__(kPrepThreads) delta_chunk_kernel(const DeltaArgs a, const Rows rows) {
  extern __shared__ __align__(16) unsigned char raw[];
  PrepSmem<D>& sm = *reinterpret_cast<PrepSmem<D>*>(raw);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int c0 = blockIdx.x * kChunk, h = blockIdx.y, kh = h / (a.heads / a.kv_heads), n = min(kChunk, rows.n - c0), ns = a.scalar_count();
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(a.qkv) + (int64_t)c0 * a.ldc + kh * D;
  for (int i = tid; i < kChunk * (D / 8); i += kPrepThreads) {
    const int r = i / (D / 8), c = i % (D / 8) * 8;
    const __nv_bfloat16* p = x + (int64_t)(r < n ? r : 0) * a.ldc + c;
    cp16_zfill(&sm.q[r][c], p, r < n);
    cp16_zfill(&sm.k[r][c], p + a.kv_heads * D, r < n);
  }
  asm volatile("cp.async.commit_group;\n" ::: "memory");
  if (warp == 0) {
    // two neighbouring rows per lane
    float lg[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = 2 * lane + e;
      const float* s = a.scalars + (int64_t)(c0 + (r < n ? r : 0)) * ns;
      sm.rq[r] = r < n ? s[kh] : 0.0f;
      sm.rk[r] = r < n ? s[a.kv_heads + kh] : 0.0f;
      sm.beta[r] = r < n ? s[2 * a.kv_heads + h] : 0.0f;
      lg[e] = r < n ? s[2 * a.kv_heads + a.heads + h] : 0.0f;
    }
    float sum = lg[0] + lg[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += up;
    }
    sm.G[2 * lane] = sum - lg[1];
    sm.G[2 * lane + 1] = sum;
  }
  asm volatile("cp.async.wait_group 0;\n" ::: "memory");
  __syncthreads();
  uint32_t* out = reinterpret_cast<uint32_t*>(a.chunks) + ((int64_t)blockIdx.x * a.heads + h) * kChunkWords;
  if (tid < kChunk) {
    const float last = sm.G[kChunk - 1], G = sm.G[tid], rk = sm.rk[tid];   // rows past the end add nothing to the sum
    float* f = reinterpret_cast<float*>(out + kFactorsAt);
    f[F_KEY + tid] = expf(G) * rk;
    f[F_QUERY + tid] = expf(G) * sm.rq[tid];
    f[F_BETA + tid] = sm.beta[tid];
    f[F_STATE + tid] = expf(last - G) * rk;
    if (tid < 4) f[F_LAST + tid] = expf(last);
  }
  const int r0 = 16 * warp;
  float kk[kChunk / 8][4] = {}, qk[kChunk / 8][4] = {};
#pragma unroll
  for (int s = 0; s < D / 16; ++s) {
    uint32_t qa[4], ka[4];
    ldsm(qa, &sm.q[r0 + (lane & 15)][16 * s + (lane >> 4) * 8]);
    ldsm(ka, &sm.k[r0 + (lane & 15)][16 * s + (lane >> 4) * 8]);
#pragma unroll
    for (int kt = 0; kt < kChunk / 16; ++kt) {
      if (kt > warp) break;
      uint32_t b[4];
      ldsm(b, &sm.k[16 * kt + (lane & 7) + (lane >> 4) * 8][16 * s + ((lane >> 3) & 1) * 8]);
      mma_bf16_16816(kk[2 * kt], ka, b[0], b[1]);
      mma_bf16_16816(kk[2 * kt + 1], ka, b[2], b[3]);
      mma_bf16_16816(qk[2 * kt], qa, b[0], b[1]);
      mma_bf16_16816(qk[2 * kt + 1], qa, b[2], b[3]);
    }
  }
#pragma unroll
  for (int nt = 0; nt < kChunk / 8; ++nt)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = r0 + g + 8 * half, j = 8 * nt + 2 * t;
      float A[2] = {}, P[2] = {};
      if (nt / 2 <= warp) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float w = j + e <= i ? expf(sm.G[i] - sm.G[j + e]) * sm.rk[j + e] : 0.0f;
          P[e] = w * sm.rq[i] * qk[nt][2 * half + e];
          A[e] = j + e < i ? w * sm.beta[i] * sm.rk[i] * kk[nt][2 * half + e] : 0.0f;
        }
        *reinterpret_cast<uint2*>(out + kChunk * kChunk + i * kChunk + j) = pack_pair(P[0], P[1]);
      }
      *reinterpret_cast<float2*>(&sm.A[i][j]) = make_float2(A[0], A[1]);
    }
  __syncthreads();
  if (tid >= kChunk) return;
  // column tid of T: T_i = e_i - sum_(j<i) A_ij T_j
  float T[kChunk];
#pragma unroll
  for (int i = 0; i < kChunk; ++i) {
    float s[4] = {i == tid ? 1.0f : 0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
    for (int j = 0; j < i; j += 4) {
      const float4 A = *reinterpret_cast<const float4*>(&sm.A[i][j]);
      s[0] = fmaf(-A.x, T[j], s[0]);
      if (j + 1 < i) s[1] = fmaf(-A.y, T[j + 1], s[1]);
      if (j + 2 < i) s[2] = fmaf(-A.z, T[j + 2], s[2]);
      if (j + 3 < i) s[3] = fmaf(-A.w, T[j + 3], s[3]);
    }
    T[i] = (s[0] + s[1]) + (s[2] + s[3]);
    const __nv_bfloat16 hi = __float2bfloat16_rn(T[i]), lo = __float2bfloat16_rn(T[i] - __bfloat162float(hi));
    out[i * kChunk + tid] = (uint32_t)__bfloat16_as_ushort(hi) | (uint32_t)__bfloat16_as_ushort(lo) << 16;
  }
}

template <int D, int VS>
struct ScanSmem {
  static constexpr int kRow = D + 8, kVRow = VS + 8, kPRow = kChunk + 4;
  __nv_bfloat16 q[2][kChunk][kRow], k[2][kChunk][kRow], v[2][kChunk][kVRow];
  uint32_t T[2][kChunk][kPRow], P[2][kChunk][kPRow];
  float f[2][F_COUNT];
  __nv_bfloat16 s_hi[D][kVRow], s_lo[D][kVRow];       // state
  __nv_bfloat16 r_hi[kChunk][kVRow], r_lo[kChunk][kVRow];
  __nv_bfloat16 u_hi[kChunk][kVRow], u_lo[kChunk][kVRow];
  __nv_bfloat16 d_hi[kChunk][kVRow], d_lo[kChunk][kVRow];   // u scaled for the state
};

// grid (heads, blocks of VS value columns).  A warp = 16 rows of a chunk x 16 columns, and every fourth 16-row tile of the
// state x the same columns, which stays in accumulator fragments between the chunks
template <int D, int VS>
__global__ void __launch_bounds__(8 * VS) delta_scan_kernel(const DeltaArgs a, const Rows rows) {
  extern __shared__ __align__(16) unsigned char raw[];
  using Smem = ScanSmem<D, VS>;
  Smem& sm = *reinterpret_cast<Smem*>(raw);
  constexpr int kScanThreads = 8 * VS, KS = D / 16, MT = (KS + 3) / 4;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int rt = warp & 3, r0 = 16 * rt, n0 = 16 * (warp >> 2);
  const int h = blockIdx.x, kh = h / (a.heads / a.kv_heads), v0 = blockIdx.y * VS;
  float* state = a.state + ((int64_t)rows.seq0 * a.heads + h) * D * a.vdim;
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(a.qkv);
  const __nv_bfloat16 *xq = x + kh * D, *xk = x + (a.kv_heads + kh) * D, *xv = x + 2 * a.kv_heads * D + h * a.vdim + v0;

  auto issue = [&](int chunk, int buf) {
    const int c0 = chunk * kChunk, n = min(kChunk, rows.n - c0);
    for (int i = tid; i < kChunk * (D / 8); i += kScanThreads) {
      const int r = i / (D / 8), c = i % (D / 8) * 8;
      const int64_t at = (int64_t)(r < n ? c0 + r : 0) * a.ldc + c;
      cp16_zfill(&sm.q[buf][r][c], xq + at, r < n);
      cp16_zfill(&sm.k[buf][r][c], xk + at, r < n);
    }
    for (int i = tid; i < kChunk * (VS / 8); i += kScanThreads) {
      const int r = i / (VS / 8), c = i % (VS / 8) * 8;
      const bool live = r < n && v0 + c < a.vdim;
      cp16_zfill(&sm.v[buf][r][c], live ? xv + (int64_t)(c0 + r) * a.ldc + c : xq, live);
    }
    const uint32_t* w = reinterpret_cast<const uint32_t*>(a.chunks) + ((int64_t)chunk * a.heads + h) * kChunkWords;
    for (int i = tid; i < kChunk * (kChunk / 4); i += kScanThreads) {
      const int r = i / (kChunk / 4), c = i % (kChunk / 4) * 4;
      if (c >= 16 * (r / 16 + 1)) continue;   // above the diagonal tiles
      cp16_zfill(&sm.T[buf][r][c], w + r * kChunk + c, true);
      cp16_zfill(&sm.P[buf][r][c], w + kChunk * kChunk + r * kChunk + c, true);
    }
    for (int i = tid; i < F_COUNT / 4; i += kScanThreads) cp16_zfill(&sm.f[buf][4 * i], w + kFactorsAt + 4 * i, true);
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  issue(0, 0);

  // state rows 16 (rt + 4 mt) + g (+8), columns n0 + 8 nt + 2t (+1)
  float S[MT][2][4];
  const bool carried = rows.pos[0] > 0;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = 16 * (rt + 4 * mt) + g + 8 * (e >> 1), c = v0 + n0 + 8 * nt + 2 * t + (e & 1);
        S[mt][nt][e] = carried && r < D && c < a.vdim ? state[(int64_t)r * a.vdim + c] : 0.0f;
      }
  auto store2 = [&](__nv_bfloat16* hi, __nv_bfloat16* lo, float p, float q) {
    uint32_t h2, l2;
    split2(p, q, h2, l2);
    *reinterpret_cast<uint32_t*>(hi) = h2;
    *reinterpret_cast<uint32_t*>(lo) = l2;
  };
  auto publish = [&]() {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      if (rt + 4 * mt >= KS) continue;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = 16 * (rt + 4 * mt) + g + 8 * half, c = n0 + 8 * nt + 2 * t;
          store2(&sm.s_hi[r][c], &sm.s_lo[r][c], S[mt][nt][2 * half], S[mt][nt][2 * half + 1]);
        }
    }
  };
  publish();

  const int chunks = (rows.n + kChunk - 1) / kChunk;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const int buf = chunk & 1, c0 = chunk * kChunk, n = min(kChunk, rows.n - c0);
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();   // this chunk has landed, the state is published, every warp is done with the chunk before
    if (chunk + 1 < chunks) issue(chunk + 1, buf ^ 1);
    const float* f = sm.f[buf];
    float o[2][4] = {};
    {
      float ks[2][4] = {};
#pragma unroll
      for (int kk = 0; kk < KS; ++kk) {
        uint32_t qa[4], ka[4], b[4];
        ldsm(qa, &sm.q[buf][r0 + (lane & 15)][16 * kk + (lane >> 4) * 8]);
        ldsm(ka, &sm.k[buf][r0 + (lane & 15)][16 * kk + (lane >> 4) * 8]);
        ldsm_trans(b, &sm.s_hi[16 * kk + (lane & 15)][n0 + (lane >> 4) * 8]);
        mma_bf16_16816(ks[0], ka, b[0], b[1]);
        mma_bf16_16816(ks[1], ka, b[2], b[3]);
        mma_bf16_16816(o[0], qa, b[0], b[1]);
        mma_bf16_16816(o[1], qa, b[2], b[3]);
        ldsm_trans(b, &sm.s_lo[16 * kk + (lane & 15)][n0 + (lane >> 4) * 8]);
        mma_bf16_16816(ks[0], ka, b[0], b[1]);
        mma_bf16_16816(ks[1], ka, b[2], b[3]);
        mma_bf16_16816(o[0], qa, b[0], b[1]);
        mma_bf16_16816(o[1], qa, b[2], b[3]);
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = r0 + g + 8 * half;
        const float beta = f[F_BETA + i], key = f[F_KEY + i], query = f[F_QUERY + i];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const int c = n0 + 8 * nt + 2 * t;
          const float2 v = unpack2(*reinterpret_cast<const uint32_t*>(&sm.v[buf][i][c]));
          store2(&sm.r_hi[i][c], &sm.r_lo[i][c], beta * (v.x - key * ks[nt][2 * half]), beta * (v.y - key * ks[nt][2 * half + 1]));
          o[nt][2 * half] *= query;
          o[nt][2 * half + 1] *= query;
        }
      }
    }
    __syncthreads();
    {
      float u[2][4] = {};
#pragma unroll
      for (int kt = 0; kt < kChunk / 16; ++kt) {
        if (kt > rt) break;
        uint32_t hi[4], lo[4], b[4];
        load_packed<Smem::kPRow>(sm.T[buf], r0, 16 * kt, hi, lo);
        ldsm_trans(b, &sm.r_hi[16 * kt + (lane & 15)][n0 + (lane >> 4) * 8]);
        mma_bf16_16816(u[0], hi, b[0], b[1]);
        mma_bf16_16816(u[1], hi, b[2], b[3]);
        mma_bf16_16816(u[0], lo, b[0], b[1]);
        mma_bf16_16816(u[1], lo, b[2], b[3]);
        ldsm_trans(b, &sm.r_lo[16 * kt + (lane & 15)][n0 + (lane >> 4) * 8]);
        mma_bf16_16816(u[0], hi, b[0], b[1]);
        mma_bf16_16816(u[1], hi, b[2], b[3]);
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = r0 + g + 8 * half;
        const float w = f[F_STATE + i];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const int c = n0 + 8 * nt + 2 * t;
          store2(&sm.u_hi[i][c], &sm.u_lo[i][c], u[nt][2 * half], u[nt][2 * half + 1]);
          store2(&sm.d_hi[i][c], &sm.d_lo[i][c], w * u[nt][2 * half], w * u[nt][2 * half + 1]);
        }
      }
    }
    __syncthreads();
    {
      const float last = f[F_LAST];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[mt][nt][e] *= last;
#pragma unroll
      for (int kt = 0; kt < kChunk / 16; ++kt) {
        if (16 * kt >= n) break;
        uint32_t bh[4], bl[4];
        ldsm_trans(bh, &sm.d_hi[16 * kt + (lane & 15)][n0 + (lane >> 4) * 8]);
        ldsm_trans(bl, &sm.d_lo[16 * kt + (lane & 15)][n0 + (lane >> 4) * 8]);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          if (rt + 4 * mt >= KS) continue;
          uint32_t ka[4];
          ldsm_trans(ka, &sm.k[buf][16 * kt + (lane & 7) + (lane >> 4) * 8][16 * (rt + 4 * mt) + ((lane >> 3) & 1) * 8]);
          mma_bf16_16816(S[mt][0], ka, bh[0], bh[1]);
          mma_bf16_16816(S[mt][1], ka, bh[2], bh[3]);
          mma_bf16_16816(S[mt][0], ka, bl[0], bl[1]);
          mma_bf16_16816(S[mt][1], ka, bl[2], bl[3]);
        }
      }
      publish();   // the old state was last read before the chunk's second barrier
    }
    // outputs
#pragma unroll
    for (int kt = 0; kt < kChunk / 16; ++kt) {
      if (kt > rt) break;
      uint32_t hi[4], lo[4], b[4];
      load_packed<Smem::kPRow>(sm.P[buf], r0, 16 * kt, hi, lo);
      ldsm_trans(b, &sm.u_hi[16 * kt + (lane & 15)][n0 + (lane >> 4) * 8]);
      mma_bf16_16816(o[0], hi, b[0], b[1]);
      mma_bf16_16816(o[1], hi, b[2], b[3]);
      mma_bf16_16816(o[0], lo, b[0], b[1]);
      mma_bf16_16816(o[1], lo, b[2], b[3]);
      ldsm_trans(b, &sm.u_lo[16 * kt + (lane & 15)][n0 + (lane >> 4) * 8]);
      mma_bf16_16816(o[0], hi, b[0], b[1]);
      mma_bf16_16816(o[1], hi, b[2], b[3]);
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = r0 + g + 8 * half;
      if (i >= n) continue;
      float* out = a.o + ((int64_t)(c0 + i) * a.heads + h) * a.vdim + v0;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        const int c = n0 + 8 * nt + 2 * t;
        if (v0 + c < a.vdim) *reinterpret_cast<float2*>(out + c) = make_float2(o[nt][2 * half], o[nt][2 * half + 1]);
      }
    }
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = 16 * (rt + 4 * mt) + g + 8 * (e >> 1), c = v0 + n0 + 8 * nt + 2 * t + (e & 1);
        if (r < D && c < a.vdim) state[(int64_t)r * a.vdim + c] = S[mt][nt][e];
      }
}

template <int D, int VS>
cudaError_t launch_scan(const DeltaArgs& a, const Rows& rows, cudaStream_t st) {
  const int smem = (int)sizeof(ScanSmem<D, VS>);
  static_assert(sizeof(ScanSmem<D, VS>) <= 227 * 1024, "shared memory of one block");
  const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<D, VS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  delta_scan_kernel<D, VS><<<dim3(a.heads, (a.vdim + VS - 1) / VS), 8 * VS, smem, st>>>(a, rows);
  return cudaGetLastError();
}
template <int D>
cudaError_t launch_chunks(const DeltaArgs& a, const Rows& rows, int sm_count, cudaStream_t st) {
  const int smem = (int)sizeof(PrepSmem<D>);
  const cudaError_t e = cudaFuncSetAttribute(delta_chunk_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  delta_chunk_kernel<D><<<dim3((rows.n + kChunk - 1) / kChunk, a.heads), kPrepThreads, smem, st>>>(a, rows);
  const cudaError_t e2 = cudaGetLastError();
  if (e2 != cudaSuccess) return e2;
  // narrower blocks where that still leaves one per SM
  return a.heads * ((a.vdim + 15) / 16) <= sm_count ? launch_scan<D, 16>(a, rows, st) : launch_scan<D, 32>(a, rows, st);
}

// a warp per (row, head)
template <class T>
__global__ void __launch_bounds__(kConvThreads) delta_norm_kernel(const DeltaArgs a, const Rows rows, T* __restrict__ out, int64_t ldo) {
  const int64_t task = (int64_t)blockIdx.x * (kConvThreads / 32) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (task >= (int64_t)rows.n * a.heads) return;
  const int64_t r = task / a.heads;
  const int h = (int)(task % a.heads);
  const float* o = a.o + task * a.vdim;
  const T* gate = static_cast<const T*>(a.proj) + r * a.ldp + a.channels() + h * a.vdim;
  float ss = 0.0f;
  for (int c = lane; c < a.vdim; c += 32) ss = fmaf(o[c], o[c], ss);
  const float inv = 1.0f / sqrtf(warp_sum(ss) / a.vdim + a.eps);
  for (int c = lane; c < a.vdim; c += 32) out[r * ldo + h * a.vdim + c] = to<T>(o[c] * inv * a.norm[c] * siluf_(from(gate[c])));
}

// heads of at most 128 values, a multiple of 4: four of them per warp, every load requested at once
constexpr int kNormHeads = 4;
template <class T>
__global__ void __launch_bounds__(kConvThreads) delta_norm_small_kernel(const DeltaArgs a, const Rows rows, T* __restrict__ out, int64_t ldo) {
  const unsigned tasks = (unsigned)rows.n * a.heads, first = (blockIdx.x * (kConvThreads / 32) + (threadIdx.x >> 5)) * kNormHeads;
  const int c = 4 * (threadIdx.x & 31);
  const bool live = c < a.vdim;
  float x[kNormHeads][4] = {}, z[kNormHeads][4] = {}, w[4] = {};
  int64_t dst[kNormHeads];
  if (live) Vec<float, 4>::load(a.norm + c, w);
#pragma unroll
  for (int i = 0; i < kNormHeads; ++i) {
    const unsigned task = first + i, r = task / (unsigned)a.heads, h = task - r * a.heads;
    dst[i] = r * ldo + h * a.vdim + c;
    if (task >= tasks || !live) continue;
    Vec<float, 4>::load(a.o + (int64_t)task * a.vdim + c, x[i]);
    Vec<T, 4>::load(static_cast<const T*>(a.proj) + r * a.ldp + a.channels() + h * a.vdim + c, z[i]);
  }
#pragma unroll
  for (int i = 0; i < kNormHeads; ++i) {
    float ss = 0.0f;
#pragma unroll
    for (int e = 0; e < 4; ++e) ss = fmaf(x[i][e], x[i][e], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / a.vdim + a.eps);
    if (first + i >= tasks || !live) continue;
#pragma unroll
    for (int e = 0; e < 4; ++e) x[i][e] = x[i][e] * inv * w[e] * siluf_(z[i][e]);
    Vec<T, 4>::store(out + dst[i], x[i]);
  }
}

}  // namespace

bool delta_chunks_supported(const DeltaArgs& a) { return a.dim % 16 == 0 && a.dim <= 128 && a.vdim % 8 == 0 && a.ldc % 8 == 0 && a.chunks; }
size_t delta_chunk_floats() { return kChunkWords; }
int delta_chunks(int rows) { return (rows + kChunk - 1) / kChunk; }

template <class TP, class TO>
cudaError_t launch_delta_step(const DeltaArgs& a, const Rows& rows, TO* out, int64_t ldo, bool pdl, cudaStream_t st) {
  const int tiles = (a.vdim + kTileCols - 1) / kTileCols;
  if (a.dim > kTileGroups * kTileRows || tiles > kMaxTiles) {
    const size_t smem = 4 * (2 * (size_t)a.dim + a.vdim + 2 * kStepGroups * kStepCols);
    if (smem > 48 * 1024) return cudaErrorInvalidValue;
    return launch_kernel(delta_step_wide_kernel<TP, TO>, dim3(a.heads, rows.n), dim3(kStepThreads), smem, st, pdl, a, rows, out, ldo);
  }
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(tiles, a.heads, rows.n);
  cfg.blockDim = dim3(kTileThreads);
  cfg.dynamicSmemBytes = 4 * (2 * (size_t)a.dim + kTileCols);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = tiles;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, delta_step_kernel<TP, TO>, a, rows, out, ldo);
}
template cudaError_t launch_delta_step<float, float>(const DeltaArgs&, const Rows&, float*, int64_t, bool, cudaStream_t);
template cudaError_t launch_delta_step<__nv_bfloat16, __nv_bfloat16>(const DeltaArgs&, const Rows&, __nv_bfloat16*, int64_t, bool, cudaStream_t);

template <class T>
cudaError_t launch_delta_prompt(const DeltaArgs& a, const Rows& rows, T* out, int64_t ldo, int sm_count, cudaStream_t st, int* launches) {
  const int tasks = 2 * a.kv_heads + a.heads + 1, warps = kConvThreads / 32;
  const dim3 grid((tasks + warps - 1) / warps, (rows.n + kConvRows - 1) / kConvRows);
  const bool few = a.taps <= 4;
  if (a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ldp % 4 == 0 && a.ldc % 4 == 0) {
    if (few) delta_conv_kernel<T, 4, true><<<grid, kConvThreads, 0, st>>>(a, rows);
    else delta_conv_kernel<T, 4, false><<<grid, kConvThreads, 0, st>>>(a, rows);
  } else {
    if (few) delta_conv_kernel<T, 1, true><<<grid, kConvThreads, 0, st>>>(a, rows);
    else delta_conv_kernel<T, 1, false><<<grid, kConvThreads, 0, st>>>(a, rows);
  }
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return e;
  delta_ring_kernel<T><<<(a.channels() + kConvThreads - 1) / kConvThreads, kConvThreads, 0, st>>>(a, rows);
  if ((e = cudaGetLastError()) != cudaSuccess) return e;
  *launches += 4;
  if (sizeof(T) == 2 && delta_chunks_supported(a)) {
    switch (a.dim / 16) {
      case 1: e = launch_chunks<16>(a, rows, sm_count, st); break;
      case 2: e = launch_chunks<32>(a, rows, sm_count, st); break;
      case 3: e = launch_chunks<48>(a, rows, sm_count, st); break;
      case 4: e = launch_chunks<64>(a, rows, sm_count, st); break;
      case 5: e = launch_chunks<80>(a, rows, sm_count, st); break;
      case 6: e = launch_chunks<96>(a, rows, sm_count, st); break;
      case 7: e = launch_chunks<112>(a, rows, sm_count, st); break;
      default: e = launch_chunks<128>(a, rows, sm_count, st); break;
    }
    if (e != cudaSuccess) return e;
    *launches += 1;
  } else {
    const size_t smem = 4 * ((size_t)a.dim * kCols + 2 * a.dim + 3 * kGroups * kCols);
    if (smem > 200 * 1024) return cudaErrorInvalidValue;
    if (smem > 48 * 1024 && (e = cudaFuncSetAttribute(delta_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) != cudaSuccess) return e;
    delta_rows_kernel<T><<<dim3(a.heads, (a.vdim + kCols - 1) / kCols), dim3(kCols, kGroups), smem, st>>>(a, rows);
    if ((e = cudaGetLastError()) != cudaSuccess) return e;
  }
  const bool small = a.dim % 2 == 0 && a.vdim % 4 == 0 && a.vdim <= 128 && a.ldp % 4 == 0 && ldo % 4 == 0;
  const int64_t per_block = warps * (small ? kNormHeads : 1);
  const unsigned blocks = (unsigned)(((int64_t)rows.n * a.heads + per_block - 1) / per_block);
  if (small) delta_norm_small_kernel<T><<<blocks, kConvThreads, 0, st>>>(a, rows, out, ldo);
  else delta_norm_kernel<T><<<blocks, kConvThreads, 0, st>>>(a, rows, out, ldo);
  return cudaGetLastError();
}
template cudaError_t launch_delta_prompt<float>(const DeltaArgs&, const Rows&, float*, int64_t, int, cudaStream_t, int*);
template cudaError_t launch_delta_prompt<__nv_bfloat16>(const DeltaArgs&, const Rows&, __nv_bfloat16*, int64_t, int, cudaStream_t, int*);

}  // namespace emelb
