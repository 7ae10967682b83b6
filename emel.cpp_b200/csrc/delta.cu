// Gated delta rule: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q / sqrt(dim), one decay g and one step size
// beta per head and token, q and k unit vectors behind a short causal convolution and silu.  The state [dim][vdim] of a
// (sequence, head) is f32 and stays in HBM between calls; a sequence that starts at position 0 starts from zero whatever
// the memory holds.
//
// One token: everything from the projections to the gated heads is one launch, a block per (head, row).
// Prompts: convolution and the tokens' scalars; the recurrence; norm and gate.  1 / |q| and 1 / |k| stay f32 factors
// beside the convolved vectors, so that the vectors themselves can be bf16 operands.
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

// ---- one token
constexpr int kStepThreads = 512, kStepCols = 128, kStepGroups = kStepThreads / kStepCols;

// grid (heads, rows).  RPT: state rows a thread keeps in registers between its two uses (0: read twice)
template <class TP, class TO, int RPT>
__global__ void __launch_bounds__(kStepThreads) delta_step_kernel(const DeltaArgs a, const Rows rows, TO* __restrict__ out, int64_t ldo) {
  extern __shared__ float sm[];
  float* q = sm;                          // [dim]
  float* k = q + a.dim;                   // [dim]
  float* v = k + a.dim;                   // [vdim], later the outputs
  float* red = v + a.vdim;                // [2][kStepGroups][kStepCols]
  __shared__ float scal[3];               // 1 / |q| / sqrt(dim), 1 / |k|, q . k (unscaled)
  __shared__ float total[kStepThreads / 32];
  pdl_trigger();
  const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rep = a.heads / a.kv_heads, kh = h / rep, channels = a.channels();
  pdl_wait();
  const int pos = rows.prompt ? rows.pos[0] : rows.pos[r], seq = rows.prompt ? rows.seq0 : rows.seq0 + r;
  const int cols = tid % kStepCols, group = tid / kStepCols;
  float* state = a.state + ((int64_t)seq * a.heads + h) * a.dim * a.vdim;
  // the state's first tile is on its way while the convolution runs
  float S[RPT > 0 ? RPT : 1];
  auto fetch = [&](int c) {
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int row = group + i * kStepGroups;
      S[i] = pos > 0 && row < a.dim && c < a.vdim ? state[(int64_t)row * a.vdim + c] : 0.0f;
    }
  };
  if (RPT > 0) fetch(cols);

  const TP* x = static_cast<const TP*>(a.proj) + (int64_t)r * a.ldp;
  float* ring = a.conv_state + (int64_t)seq * a.taps * channels;
  for (int i = tid; i < 2 * a.dim + a.vdim; i += kStepThreads) {
    const int c = i < a.dim ? kh * a.dim + i : i < 2 * a.dim ? (a.kv_heads + kh) * a.dim + i - a.dim : 2 * a.kv_heads * a.dim + h * a.vdim + i - 2 * a.dim;
    const float u = from(x[c]);
    float y = a.conv[(int64_t)(a.taps - 1) * channels + c] * u;
    for (int b = 1; b < a.taps && b <= pos; ++b) y = fmaf(a.conv[(int64_t)(a.taps - 1 - b) * channels + c], ring[(int64_t)((pos - b) % a.taps) * channels + c], y);
    // no block reads this entry in this step: its old token lies `taps` back
    if (i >= 2 * a.dim || h % rep == 0) ring[(int64_t)(pos % a.taps) * channels + c] = u;
    sm[i] = siluf_(y);
  }
  __syncthreads();
  if (warp < 3) {
    const float *s0 = warp == 1 ? k : q, *s1 = warp == 0 ? q : k;
    float s = 0.0f;
    for (int i = lane; i < a.dim; i += 32) s = fmaf(s0[i], s1[i], s);
    s = warp_sum(s);
    if (lane == 0) scal[warp] = warp == 2 ? s : 1.0f / sqrtf(s + kUnitEps) * (warp == 0 ? 1.0f / sqrtf((float)a.dim) : 1.0f);
  }
  const float* gates = a.gates + (int64_t)r * a.ldg;
  const float beta = sigmoidf_(gates[h]), g = expf(log_decay(a, h, gates[a.heads + h]));
  __syncthreads();
  const float rq = scal[0], rk = scal[1], qk = scal[2] * rq * rk;

  float ss = 0.0f;
  for (int c0 = 0; c0 < a.vdim; c0 += kStepCols) {
    const int c = c0 + cols;
    const bool live = c < a.vdim;
    if (RPT > 0 && c0 > 0) fetch(c);
    float sk = 0.0f, sq = 0.0f;
    if (RPT > 0) {
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        const int row = group + i * kStepGroups;
        if (row < a.dim) {
          sk = fmaf(S[i], k[row], sk);
          sq = fmaf(S[i], q[row], sq);
        }
      }
    } else if (live && pos > 0) {
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
      const float ku = rk * u;
      if (RPT > 0) {
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
          const int row = group + i * kStepGroups;
          if (row < a.dim) state[(int64_t)row * a.vdim + c] = fmaf(k[row], ku, g * S[i]);
        }
      } else {
#pragma unroll 8
        for (int row = group; row < a.dim; row += kStepGroups) {
          const float s = pos > 0 ? state[(int64_t)row * a.vdim + c] : 0.0f;
          state[(int64_t)row * a.vdim + c] = fmaf(k[row], ku, g * s);
        }
      }
      if (group == 0) {
        v[c] = o;
        ss = fmaf(o, o, ss);
      }
    }
  }
  ss = warp_sum(ss);
  if (lane == 0) total[warp] = ss;
  __syncthreads();
  ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kStepCols / 32; ++i) ss += total[i];   // the first group's warps
  const float inv = 1.0f / sqrtf(ss / a.vdim + a.eps);
  const TP* gate = x + channels + h * a.vdim;
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
template <class T, int V>
__global__ void __launch_bounds__(kConvThreads) delta_conv_kernel(const DeltaArgs a, const Rows rows) {
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
    // the input of row r meets the rows r .. r + taps - 1
    for (int r = r0 - (a.taps - 1); r < r0 + nr; ++r) {
      float u[V];
      if (r >= 0) {
        Vec<T, V>::load(proj + (int64_t)r * a.ldp + c, u);
      } else if (pos0 + r >= 0) {
        Vec<float, V>::load(ring + (int64_t)((pos0 + r) % a.taps) * channels + c, u);
      } else {
        continue;
      }
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

}  // namespace

bool delta_chunks_supported(const DeltaArgs&) { return false; }
size_t delta_chunk_floats() { return 1; }
int delta_chunks(int rows) { return (rows + 63) / 64; }

template <class TP, class TO>
cudaError_t launch_delta_step(const DeltaArgs& a, const Rows& rows, TO* out, int64_t ldo, bool pdl, cudaStream_t st) {
  const size_t smem = 4 * (2 * (size_t)a.dim + a.vdim + 2 * kStepGroups * kStepCols);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  auto kern = a.dim <= 32 * kStepGroups ? delta_step_kernel<TP, TO, 32> : delta_step_kernel<TP, TO, 0>;
  return launch_kernel(kern, dim3(a.heads, rows.n), dim3(kStepThreads), smem, st, pdl, a, rows, out, ldo);
}
template cudaError_t launch_delta_step<float, float>(const DeltaArgs&, const Rows&, float*, int64_t, bool, cudaStream_t);
template cudaError_t launch_delta_step<__nv_bfloat16, __nv_bfloat16>(const DeltaArgs&, const Rows&, __nv_bfloat16*, int64_t, bool, cudaStream_t);

template <class T>
cudaError_t launch_delta_prompt(const DeltaArgs& a, const Rows& rows, T* out, int64_t ldo, cudaStream_t st, int* launches) {
  const int tasks = 2 * a.kv_heads + a.heads + 1, warps = kConvThreads / 32;
  const dim3 grid((tasks + warps - 1) / warps, (rows.n + kConvRows - 1) / kConvRows);
  if (a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ldp % 4 == 0 && a.ldc % 4 == 0) delta_conv_kernel<T, 4><<<grid, kConvThreads, 0, st>>>(a, rows);
  else delta_conv_kernel<T, 1><<<grid, kConvThreads, 0, st>>>(a, rows);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return e;
  delta_ring_kernel<T><<<(a.channels() + kConvThreads - 1) / kConvThreads, kConvThreads, 0, st>>>(a, rows);
  if ((e = cudaGetLastError()) != cudaSuccess) return e;
  const size_t smem = 4 * ((size_t)a.dim * kCols + 2 * a.dim + 3 * kGroups * kCols);
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  if (smem > 48 * 1024 && (e = cudaFuncSetAttribute(delta_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) != cudaSuccess) return e;
  delta_rows_kernel<T><<<dim3(a.heads, (a.vdim + kCols - 1) / kCols), dim3(kCols, kGroups), smem, st>>>(a, rows);
  if ((e = cudaGetLastError()) != cudaSuccess) return e;
  delta_norm_kernel<T><<<(unsigned)(((int64_t)rows.n * a.heads + warps - 1) / warps), kConvThreads, 0, st>>>(a, rows, out, ldo);
  *launches += 4;
  return cudaGetLastError();
}
template cudaError_t launch_delta_prompt<float>(const DeltaArgs&, const Rows&, float*, int64_t, cudaStream_t, int*);
template cudaError_t launch_delta_prompt<__nv_bfloat16>(const DeltaArgs&, const Rows&, __nv_bfloat16*, int64_t, cudaStream_t, int*);

}  // namespace emelb
