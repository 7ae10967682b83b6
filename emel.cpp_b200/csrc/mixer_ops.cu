// Row kernels of layered decoders between the products: embedding, residual + norm, gated RMS norm, GLU, and the
// step from an attention layer's projections to its queries and cache rows (short convolution, query / key norm over
// the whole projection, partial rotation, value norm, store).  f32 arithmetic throughout.
#include <math.h>

#include "act.cuh"
#include "common.cuh"
#include "layered.h"

namespace emelb {
namespace {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;

template <class T>
__device__ __forceinline__ T to(float x);
template <>
__device__ __forceinline__ float to<float>(float x) { return x; }
template <>
__device__ __forceinline__ __nv_bfloat16 to<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }
__device__ __forceinline__ float from(float x) { return x; }
__device__ __forceinline__ float from(__nv_bfloat16 x) { return __bfloat162float(x); }

template <int WARPS = kWarps>
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.0f;
#pragma unroll
  for (int w = 0; w < WARPS; ++w) t += scratch[w];
  return t;
}

__device__ __forceinline__ void store_pair(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }

template <class T>
__global__ void embed_rows_bf16_kernel(const __nv_bfloat16* __restrict__ table, int64_t ld, const int* __restrict__ tokens,
                                       const float* __restrict__ step, int width, float* x, T* xb, int64_t ldb) {
  const int r = blockIdx.x;
  const __nv_bfloat16* row = table + (int64_t)tokens[r] * ld;
  for (int i = threadIdx.x; i < width; i += kThreads) {
    const float v = __bfloat162float(row[i]) + (step ? step[i] : 0.0f);
    x[(int64_t)r * width + i] = v;
    xb[(int64_t)r * ldb + i] = to<T>(v);
  }
}

// norm of the vector in shared memory: mean (0 for an RMS norm) and 1 / sqrt(mean square of the deviations + eps),
// the deviations in a second pass
__device__ __forceinline__ void norm_stats(const float* s, int n, int rms, float eps, float* scratch, float& mean, float& inv) {
  float t = 0.0f;
  mean = 0.0f;
  if (!rms) {
    for (int i = threadIdx.x; i < n; i += kThreads) t += s[i];
    mean = block_sum(t, scratch) / n;
  }
  t = 0.0f;
  for (int i = threadIdx.x; i < n; i += kThreads) {
    const float d = s[i] - mean;
    t = fmaf(d, d, t);
  }
  inv = 1.0f / sqrtf(block_sum(t, scratch) / n + eps);
}

template <class T>
__global__ void residual_norm_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w, int rms, float eps,
                                     int width, T* __restrict__ xb, int64_t ldb, float* keep, const float* __restrict__ step) {
  extern __shared__ float s[];
  __shared__ float scratch[kWarps];
  const int64_t r = blockIdx.x;
  for (int i = threadIdx.x; i < width; i += kThreads) s[i] = y[r * width + i];
  float mean, inv;
  norm_stats(s, width, rms, eps, scratch, mean, inv);
  for (int i = threadIdx.x; i < width; i += kThreads) {
    float v = x[r * width + i] + (s[i] - mean) * inv * w[i];
    if (keep) keep[r * width + i] = v;
    if (step) v += step[i];
    x[r * width + i] = v;
    xb[r * ldb + i] = to<T>(v);
  }
}

template <class T>
__global__ void norm_rows_kernel(const float* __restrict__ x, const int* __restrict__ index, const float* __restrict__ w, int rms, float eps, int width,
                                 T* __restrict__ out, int64_t ldo) {
  extern __shared__ float s[];
  __shared__ float scratch[kWarps];
  const int64_t r = blockIdx.x, src = index ? index[r] : r;
  for (int i = threadIdx.x; i < width; i += kThreads) s[i] = x[src * width + i];
  float mean, inv;
  norm_stats(s, width, rms, eps, scratch, mean, inv);
  for (int i = threadIdx.x; i < width; i += kThreads) out[r * ldo + i] = to<T>((s[i] - mean) * inv * w[i]);
}

template <class T>
__global__ void prenorm_rows_kernel(const PrenormArgs a) {
  extern __shared__ float s[];
  __shared__ float scratch[kWarps];
  const int64_t r = blockIdx.x;
  const __nv_bfloat16* row = a.table ? a.table + (int64_t)a.tokens[r] * a.table_ld : nullptr;
  for (int i = threadIdx.x; i < a.width; i += kThreads) {
    float v = row ? __bfloat162float(row[i]) : a.x[r * a.width + i];
    if (a.y) v += a.y[r * a.width + i];
    if (a.keep) a.keep[r * a.width + i] = v;
    if (a.step) v += a.step[i];
    a.x[r * a.width + i] = v;
    s[i] = v;
  }
  if (!a.h1 && !a.h2) return;
  float mean, inv;
  norm_stats(s, a.width, a.rms, a.eps, scratch, mean, inv);
  for (int i = threadIdx.x; i < a.width; i += kThreads) {
    const float n = (s[i] - mean) * inv;
    if (a.h1) static_cast<T*>(a.h1)[r * a.ldh + i] = to<T>(n * a.w1[i]);
    if (a.h2) static_cast<T*>(a.h2)[r * a.ldh + i] = to<T>(n * a.w2[i]);
  }
}

template <class T>
__global__ void rms_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, const T* __restrict__ gate, int64_t ldg, float eps,
                                int width, T* __restrict__ out, int64_t ldo) {
  __shared__ float scratch[kWarps];
  const int64_t r = blockIdx.x;
  float ss = 0.0f;
  for (int i = threadIdx.x; i < width; i += kThreads) {
    const float v = o[r * width + i];
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / width + eps);
  for (int i = threadIdx.x; i < width; i += kThreads) out[r * ldo + i] = to<T>(o[r * width + i] * inv * w[i] * from(gate[r * ldg + i]));
}

__global__ void glu_rows_kernel(const float* __restrict__ gu, int ff, int act, float* __restrict__ out, int64_t ldo) {
  const int64_t r = blockIdx.y;
  const int i = blockIdx.x * kThreads + threadIdx.x;
  if (i >= ff) return;
  const float g = gu[r * 2 * ff + i], u = gu[r * 2 * ff + ff + i];
  out[r * ldo + i] = (act == ACT_GLU_GELU ? gelu_tanhf_(g) : siluf_(g)) * u;
}

// V = 1 or 4 consecutive channels
template <int V>
struct Chan { float f[V]; };
template <int V>
__device__ __forceinline__ Chan<V> load_chan(const float* p) {
  Chan<V> c;
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    c.f[0] = v.x; c.f[1] = v.y; c.f[2] = v.z; c.f[3] = v.w;
  } else {
    c.f[0] = *p;
  }
  return c;
}
template <int V>
__device__ __forceinline__ void store_chan(float* p, const Chan<V>& c) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(c.f[0], c.f[1], c.f[2], c.f[3]);
  else *p = c.f[0];
}

// One block = one row of the queries (part 0), keys (1) or values (2), V channels per thread and turn.
template <class T, int THREADS, int V>
__global__ void __launch_bounds__(THREADS) attn_in_kernel(const AttnInArgs a, const Rows rows) {
  extern __shared__ __align__(16) float s[];
  __shared__ float scratch[THREADS / 32];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, part = blockIdx.y, tid = threadIdx.x;
  const int pos = rows.prompt ? rows.pos[0] + r : rows.pos[r];
  const int seq = rows.prompt ? rows.seq0 : rows.seq0 + r;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
  const int n = part == 0 ? nq : part == 1 ? nk : nv, off = part == 0 ? 0 : part == 1 ? nq : nq + nk;
  const int hist = a.taps - 1;
  float* state = a.conv_state + (int64_t)seq * hist * a.channels;

  float ss = 0.0f;
  for (int i = tid * V; i < n; i += THREADS * V) {
    const int c = off + i;
    const Chan<V> u = load_chan<V>(a.proj + (int64_t)r * a.channels + c);
    Chan<V> y = u;
    if (a.conv) {
      const Chan<V> wl = load_chan<V>(a.conv + (int64_t)hist * a.channels + c);
#pragma unroll
      for (int e = 0; e < V; ++e) y.f[e] = wl.f[e] * u.f[e];
      for (int b = 1; b <= hist && b <= pos; ++b) {   // b tokens back
        const Chan<V> past = rows.prompt && r - b >= 0 ? load_chan<V>(a.proj + (int64_t)(r - b) * a.channels + c)
                                                       : load_chan<V>(state + (int64_t)(hist - (rows.prompt ? b - r : b)) * a.channels + c);
        const Chan<V> w = load_chan<V>(a.conv + (int64_t)(hist - b) * a.channels + c);
#pragma unroll
        for (int e = 0; e < V; ++e) y.f[e] = fmaf(w.f[e], past.f[e], y.f[e]);
      }
      if (!rows.prompt) {
        for (int j = 0; j + 1 < hist; ++j) {
          Chan<V> next = load_chan<V>(state + (int64_t)(j + 1) * a.channels + c);
          if (pos - hist + 1 + j < 0) next = Chan<V>{};
          store_chan<V>(state + (int64_t)j * a.channels + c, next);
        }
        if (hist > 0) store_chan<V>(state + (int64_t)(hist - 1) * a.channels + c, u);
      }
    }
    store_chan<V>(s + i, y);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(y.f[e], y.f[e], ss);
  }

  if (part == 2) {
    __syncthreads();
    // a warp per value head
    T* cache = static_cast<T*>(a.v);
    for (int h = tid >> 5; h < a.kv_heads; h += THREADS / 32) {
      const float* v = s + h * a.vdim;
      float inv = 1.0f;
      if (a.norm_v) {
        float t = 0.0f;
        for (int d = tid & 31; d < a.vdim; d += 32) t = fmaf(v[d], v[d], t);
        inv = 1.0f / sqrtf(warp_sum(t) / a.vdim + a.eps);
      }
      T* row = cache + (((int64_t)seq * a.kv_heads + h) * a.capacity + pos) * a.vdim_pad;
      for (int d = 2 * (tid & 31); d < a.vdim_pad; d += 64)
        store_pair(row + d, d < a.vdim ? v[d] * inv : 0.0f, d + 1 < a.vdim ? v[d + 1] * inv : 0.0f);
    }
    return;
  }
  const float* nw = part == 0 ? a.norm_q : a.norm_k;
  const float inv = 1.0f / sqrtf(block_sum<THREADS / 32>(ss, scratch) / n + a.eps);   // also orders the writes of s
  const int heads = part == 0 ? a.heads : a.kv_heads;
  auto normed = [&](int i) { return nw ? s[i] * inv * nw[i] : s[i]; };
  const int half_pad = a.dim_pad / 2;
  for (int idx = tid; idx < heads * half_pad; idx += THREADS) {
    const int h = idx / half_pad, p = idx - h * half_pad, d = 2 * p;
    float x0 = d < a.dim ? normed(h * a.dim + d) : 0.0f, x1 = d + 1 < a.dim ? normed(h * a.dim + d + 1) : 0.0f;
    if (d < a.rope_dim) {
      const int64_t t = (int64_t)pos * (a.rope_dim / 2) + p;
      const float c = a.rope_cos[t], sn = a.rope_sin[t];
      const float u = x0 * c - x1 * sn, v = x1 * c + x0 * sn;
      x0 = u;
      x1 = v;
    }
    T* row = part == 0 ? static_cast<T*>(a.q) + ((int64_t)r * a.heads + h) * a.dim_pad
                       : static_cast<T*>(a.k) + (((int64_t)seq * a.kv_heads + h) * a.capacity + pos) * a.dim_pad;
    store_pair(row + d, x0, x1);
  }
}

__global__ void conv_state_kernel(const AttnInArgs a, const Rows rows) {
  const int c = blockIdx.x * kThreads + threadIdx.x, hist = a.taps - 1;
  if (c >= a.channels) return;
  float* st = a.conv_state + (int64_t)rows.seq0 * hist * a.channels + c;
  // entry j holds the row hist - j before the next one; an old entry moves down by rows.n >= 1 places
  for (int j = 0; j < hist; ++j) {
    const int r = rows.n - hist + j;
    float v = 0.0f;
    if (r >= 0) v = a.proj[(int64_t)r * a.channels + c];
    else if (rows.pos[0] + r >= 0) v = st[(int64_t)(hist + r) * a.channels];
    st[(int64_t)j * a.channels] = v;
  }
}

}  // namespace

template <class T>
cudaError_t launch_embed_rows_bf16(const __nv_bfloat16* table, int64_t ld, const int* tokens, const float* step, int rows, int width, float* x,
                                   T* xb, int64_t ldb, cudaStream_t st) {
  embed_rows_bf16_kernel<T><<<rows, kThreads, 0, st>>>(table, ld, tokens, step, width, x, xb, ldb);
  return cudaGetLastError();
}
template cudaError_t launch_embed_rows_bf16<float>(const __nv_bfloat16*, int64_t, const int*, const float*, int, int, float*, float*, int64_t,
                                                   cudaStream_t);
template cudaError_t launch_embed_rows_bf16<__nv_bfloat16>(const __nv_bfloat16*, int64_t, const int*, const float*, int, int, float*, __nv_bfloat16*,
                                                           int64_t, cudaStream_t);

namespace {
// the same limit for every size: launches of other sizes may already be in a captured step
template <class K>
cudaError_t allow_smem(K kern, size_t bytes) {
  return bytes > 48 * 1024 ? cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) : cudaSuccess;
}
}  // namespace

template <class T>
cudaError_t launch_residual_norm(float* x, const float* y, const float* w, int rms, float eps, int rows, int width, T* xb, int64_t ldb, float* keep,
                                 const float* step, cudaStream_t st) {
  const size_t smem = 4 * (size_t)width;
  const cudaError_t e = allow_smem(residual_norm_kernel<T>, smem);
  if (e != cudaSuccess) return e;
  residual_norm_kernel<T><<<rows, kThreads, smem, st>>>(x, y, w, rms, eps, width, xb, ldb, keep, step);
  return cudaGetLastError();
}
template cudaError_t launch_residual_norm<float>(float*, const float*, const float*, int, float, int, int, float*, int64_t, float*, const float*,
                                                 cudaStream_t);
template cudaError_t launch_residual_norm<__nv_bfloat16>(float*, const float*, const float*, int, float, int, int, __nv_bfloat16*, int64_t, float*,
                                                         const float*, cudaStream_t);

template <class T>
cudaError_t launch_norm_rows(const float* x, const int* index, const float* w, int rms, float eps, int rows, int width, T* out, int64_t ldo,
                             cudaStream_t st) {
  const size_t smem = 4 * (size_t)width;
  const cudaError_t e = allow_smem(norm_rows_kernel<T>, smem);
  if (e != cudaSuccess) return e;
  norm_rows_kernel<T><<<rows, kThreads, smem, st>>>(x, index, w, rms, eps, width, out, ldo);
  return cudaGetLastError();
}
template cudaError_t launch_norm_rows<float>(const float*, const int*, const float*, int, float, int, int, float*, int64_t, cudaStream_t);
template cudaError_t launch_norm_rows<__nv_bfloat16>(const float*, const int*, const float*, int, float, int, int, __nv_bfloat16*, int64_t, cudaStream_t);

template <class T>
cudaError_t launch_prenorm_rows(const PrenormArgs& a, cudaStream_t st) {
  const size_t smem = 4 * (size_t)a.width;
  const cudaError_t e = allow_smem(prenorm_rows_kernel<T>, smem);
  if (e != cudaSuccess) return e;
  prenorm_rows_kernel<T><<<a.rows, kThreads, smem, st>>>(a);
  return cudaGetLastError();
}
template cudaError_t launch_prenorm_rows<float>(const PrenormArgs&, cudaStream_t);
template cudaError_t launch_prenorm_rows<__nv_bfloat16>(const PrenormArgs&, cudaStream_t);

template <class T>
cudaError_t launch_rms_gate(const float* o, const float* w, const T* gate, int64_t ldg, float eps, int rows, int width, T* out, int64_t ldo,
                            cudaStream_t st) {
  rms_gate_kernel<T><<<rows, kThreads, 0, st>>>(o, w, gate, ldg, eps, width, out, ldo);
  return cudaGetLastError();
}
template cudaError_t launch_rms_gate<float>(const float*, const float*, const float*, int64_t, float, int, int, float*, int64_t, cudaStream_t);
template cudaError_t launch_rms_gate<__nv_bfloat16>(const float*, const float*, const __nv_bfloat16*, int64_t, float, int, int, __nv_bfloat16*,
                                                    int64_t, cudaStream_t);

cudaError_t launch_glu_rows(const float* gu, int rows, int ff, int act, float* out, int64_t ldo, cudaStream_t st) {
  glu_rows_kernel<<<dim3((ff + kThreads - 1) / kThreads, rows), kThreads, 0, st>>>(gu, ff, act, out, ldo);
  return cudaGetLastError();
}

namespace {
template <class T, int THREADS, int V>
cudaError_t launch_attn_in_sized(const AttnInArgs& a, const Rows& rows, size_t smem, cudaStream_t st) {
  const cudaError_t e = allow_smem(attn_in_kernel<T, THREADS, V>, smem);
  if (e != cudaSuccess) return e;
  attn_in_kernel<T, THREADS, V><<<dim3(rows.n, a.own_kv ? 3 : 1), THREADS, smem, st>>>(a, rows);
  return cudaGetLastError();
}
}  // namespace

template <class T>
cudaError_t launch_attn_in(const AttnInArgs& a, const Rows& rows, cudaStream_t st) {
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
  const size_t smem = 4 * (size_t)(a.own_kv && nv > nq ? nv : nq);
  const bool quads = nq % 4 == 0 && (!a.own_kv || (nk % 4 == 0 && nv % 4 == 0));
  // few rows: a wide block each
  if (rows.n <= 16) return quads ? launch_attn_in_sized<T, 1024, 4>(a, rows, smem, st) : launch_attn_in_sized<T, 1024, 1>(a, rows, smem, st);
  return quads ? launch_attn_in_sized<T, kThreads, 4>(a, rows, smem, st) : launch_attn_in_sized<T, kThreads, 1>(a, rows, smem, st);
}
template cudaError_t launch_attn_in<float>(const AttnInArgs&, const Rows&, cudaStream_t);
template cudaError_t launch_attn_in<__nv_bfloat16>(const AttnInArgs&, const Rows&, cudaStream_t);

cudaError_t launch_conv_state(const AttnInArgs& a, const Rows& rows, cudaStream_t st) {
  conv_state_kernel<<<(a.channels + kThreads - 1) / kThreads, kThreads, 0, st>>>(a, rows);
  return cudaGetLastError();
}

}  // namespace emelb
