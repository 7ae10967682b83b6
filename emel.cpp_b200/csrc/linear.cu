// Products with bf16 weights on the CUDA cores: the one-row kernel of the decode step (streams the weights once, with
// the step before it fused into its input and the activation into its output) and a plain f32 tile kernel for many
// rows in full f32.  f32 activations and accumulation in both.
#include <cstdlib>

#include "act.cuh"
#include "common.cuh"
#include "layered.h"

namespace emelb {
namespace {

constexpr int kVecThreads = 256;
constexpr int kVecWarps = kVecThreads / 32;

__device__ __forceinline__ float block_sum(float v, float* scratch) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.0f;
#pragma unroll
  for (int w = 0; w < kVecWarps; ++w) t += scratch[w];
  return t;
}

__device__ __forceinline__ uint4 load_stream(const uint4* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// Input vector in shared memory, split so that a warp's reads of one half chunk are contiguous: elements 8c..8c+3 at
// lo[c], 8c+4..8c+7 at hi[c].
struct SplitVec {
  float* lo;
  float* hi;
  __device__ __forceinline__ float& at(int i) const { return ((i & 4) ? hi : lo)[(i >> 3) * 4 + (i & 3)]; }
  __device__ __forceinline__ float4& quad(int j) const { return *reinterpret_cast<float4*>(((j & 1) ? hi : lo) + 4 * (j >> 1)); }   // elements 4j ..
};
__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float4 scale4(float4 x, float mean, float inv, float4 w) {
  return make_float4((x.x - mean) * inv * w.x, (x.y - mean) * inv * w.y, (x.z - mean) * inv * w.z, (x.w - mean) * inv * w.w);
}
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

// A warp owns RW rows at a time (for a GLU a gate row and its up row) and walks them in 16-byte chunks, U per lane
// in flight; the first chunks are requested before the wait for the kernel in front.  DUAL: the tasks of a second matrix,
// which meets the input with the other norm weight, follow those of the first.
template <int RW, int U, bool DUAL>
__global__ void __launch_bounds__(kVecThreads, RW == 2 ? 4 : 3) linear_vec_kernel(const LinearArgs a, const VecArgs v) {
  extern __shared__ __align__(16) float xs_raw[];
  __shared__ float scratch[kVecWarps];
  pdl_trigger();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int K = a.w.K, chunks = (K + 7) / 8;
  const SplitVec xs{xs_raw, xs_raw + 4 * chunks}, xs2{xs_raw + 8 * chunks, xs_raw + 12 * chunks};
  auto glu_of = [](int act) { return act == ACT_GLU || act == ACT_GLU_GELU; };
  auto outs_of = [&](const Bf16Matrix& w, int act) { return glu_of(act) ? w.M / 2 : w.M; };
  auto tasks_of = [&](int outs, int act) { return glu_of(act) ? outs : (outs + RW - 1) / RW; };
  const int outs1 = outs_of(a.w, a.act), tasks1 = tasks_of(outs1, a.act);
  const int outs2 = DUAL ? outs_of(v.w2, v.act2) : 0;
  const int tasks = tasks1 + (DUAL ? tasks_of(outs2, v.act2) : 0);
  const int stride = gridDim.x * kVecWarps;
  int task = blockIdx.x * kVecWarps + warp;

  uint4 w[RW][U];
  auto load = [&](int t, int c0) {
    const bool second = DUAL && t >= tasks1;
    const Bf16Matrix& m = second ? v.w2 : a.w;
    const int outs = second ? outs2 : outs1, task_at = second ? t - tasks1 : t;
    const bool glu = glu_of(second ? v.act2 : a.act);
#pragma unroll
    for (int r = 0; r < RW; ++r) {
      const uint4* p = reinterpret_cast<const uint4*>(m.w + (int64_t)(glu ? task_at + r * outs : min(task_at * RW + r, outs - 1)) * m.ld);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + lane + 32 * u;
        w[r][u] = c < chunks ? load_stream(p + c) : make_uint4(0, 0, 0, 0);
      }
    }
  };
  if (task < tasks) load(task, 0);
  if (v.pro == PRO_PRENORM)
    for (int i = 32 * tid; i < K; i += 32 * kVecThreads) {
      prefetch_l2(v.norm_w + i);
      if (DUAL) prefetch_l2(v.norm2_w + i);
    }
  pdl_wait();

  // ---- the input vector
  for (int i = K + tid; i < 8 * chunks; i += kVecThreads) {
    xs.at(i) = 0.0f;
    if (DUAL) xs2.at(i) = 0.0f;
  }
  const int quads = K / 4;
  auto ld4 = [](const float* p, int j) { return reinterpret_cast<const float4*>(p)[j]; };
  if (v.pro == PRO_PLAIN) {
#pragma unroll 8
    for (int j = tid; j < quads; j += kVecThreads) xs.quad(j) = ld4(v.x, j);
    for (int i = 4 * quads + tid; i < K; i += kVecThreads) xs.at(i) = v.x[i];
  } else if (v.pro == PRO_EMBED) {
    const __nv_bfloat16* row = v.table + (int64_t)*v.token * v.table_ld;
    for (int i = tid; i < K; i += kVecThreads) {
      const float x = __bfloat162float(row[i]) + (v.step ? v.step[i] : 0.0f);
      xs.at(i) = x;
      if (blockIdx.x == 0) v.x_out[i] = x;
    }
  } else if (v.pro == PRO_PRENORM) {
    const __nv_bfloat16* row = v.table ? v.table + (int64_t)*v.token * v.table_ld : nullptr;
    float s = 0.0f, ss = 0.0f;
#pragma unroll 4
    for (int j = tid; j < quads; j += kVecThreads) {
      float4 x;
      if (row) {
        const uint2 t = reinterpret_cast<const uint2*>(row)[j];
        x = make_float4(__uint_as_float(t.x << 16), __uint_as_float(t.x & 0xffff0000u), __uint_as_float(t.y << 16), __uint_as_float(t.y & 0xffff0000u));
      } else {
        x = ld4(v.x, j);
      }
      if (v.y) x = add4(x, ld4(v.y, j));
      if (v.step) x = make_float4(x.x + v.step[4 * j], x.y + v.step[4 * j + 1], x.z + v.step[4 * j + 2], x.w + v.step[4 * j + 3]);
      xs.quad(j) = x;
      s += (x.x + x.y) + (x.z + x.w);
      ss = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, ss))));
      if (v.x_out && blockIdx.x == 0) reinterpret_cast<float4*>(v.x_out)[j] = x;
    }
    for (int i = 4 * quads + tid; i < K; i += kVecThreads) {
      float x = row ? __bfloat162float(row[i]) : v.x[i];
      if (v.y) x += v.y[i];
      if (v.step) x += v.step[i];
      xs.at(i) = x;
      s += x;
      ss = fmaf(x, x, ss);
      if (v.x_out && blockIdx.x == 0) v.x_out[i] = x;
    }
    float mean = 0.0f;
    if (!v.rms) {
      mean = block_sum(s, scratch) / K;
      ss = 0.0f;
      for (int j = tid; j < quads; j += kVecThreads) {
        const float4 x = xs.quad(j);
        ss = fmaf(x.x - mean, x.x - mean, fmaf(x.y - mean, x.y - mean, fmaf(x.z - mean, x.z - mean, fmaf(x.w - mean, x.w - mean, ss))));
      }
      for (int i = 4 * quads + tid; i < K; i += kVecThreads) ss = fmaf(xs.at(i) - mean, xs.at(i) - mean, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / K + v.eps);
#pragma unroll 4
    for (int j = tid; j < quads; j += kVecThreads) {
      const float4 x = xs.quad(j);
      xs.quad(j) = scale4(x, mean, inv, ld4(v.norm_w, j));
      if (DUAL) xs2.quad(j) = scale4(x, mean, inv, ld4(v.norm2_w, j));
    }
    for (int i = 4 * quads + tid; i < K; i += kVecThreads) {
      const float n = (xs.at(i) - mean) * inv;
      xs.at(i) = n * v.norm_w[i];
      if (DUAL) xs2.at(i) = n * v.norm2_w[i];
    }
  } else if (v.pro == PRO_RMS_GATE) {
    float ss = 0.0f;
    for (int i = tid; i < K; i += kVecThreads) {
      const float x = v.x[i];
      xs.at(i) = x;
      ss = fmaf(x, x, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / K + v.eps);
    for (int i = tid; i < K; i += kVecThreads) xs.at(i) = xs.at(i) * inv * v.norm_w[i] * v.gate[i];
  } else {
    float s = 0.0f;
    for (int i = tid; i < K; i += kVecThreads) {
      const float y = v.y[i];
      xs.at(i) = y;
      s += y;
    }
    const float mean = v.rms ? 0.0f : block_sum(s, scratch) / K;
    float ss = 0.0f;
    for (int i = tid; i < K; i += kVecThreads) {
      const float d = xs.at(i) - mean;
      ss = fmaf(d, d, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / K + v.eps);
    s = 0.0f;
    for (int i = tid; i < K; i += kVecThreads) {
      const float x = v.x[i] + (xs.at(i) - mean) * inv * v.norm_w[i] + (v.step ? v.step[i] : 0.0f);
      xs.at(i) = x;
      s += x;
      if (v.x_out && blockIdx.x == 0) v.x_out[i] = x;
    }
    if (v.pro == PRO_RESIDUAL_NORM) {
      const float mean2 = v.rms ? 0.0f : block_sum(s, scratch) / K;
      ss = 0.0f;
      for (int i = tid; i < K; i += kVecThreads) {
        const float d = xs.at(i) - mean2;
        ss = fmaf(d, d, ss);
      }
      const float inv2 = 1.0f / sqrtf(block_sum(ss, scratch) / K + v.eps);
      for (int i = tid; i < K; i += kVecThreads) xs.at(i) = (xs.at(i) - mean2) * inv2 * v.norm2_w[i];
    }
  }
  __syncthreads();

  float best = 0.0f;
  int best_row = -1;
  for (; task < tasks; task += stride) {
    const bool second = DUAL && task >= tasks1;
    const SplitVec in = second ? xs2 : xs;
    float acc[RW];
#pragma unroll
    for (int r = 0; r < RW; ++r) acc[r] = 0.0f;
    for (int c0 = 0; c0 < chunks; c0 += 32 * U) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + lane + 32 * u;
        if (c < chunks) {
          const float4 xl = *reinterpret_cast<const float4*>(in.lo + 4 * c), xh = *reinterpret_cast<const float4*>(in.hi + 4 * c);
          const float x[8] = {xl.x, xl.y, xl.z, xl.w, xh.x, xh.y, xh.z, xh.w};
#pragma unroll
          for (int r = 0; r < RW; ++r) {
            const uint32_t q[4] = {w[r][u].x, w[r][u].y, w[r][u].z, w[r][u].w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              acc[r] = fmaf(__uint_as_float(q[i] << 16), x[2 * i], acc[r]);
              acc[r] = fmaf(__uint_as_float(q[i] & 0xffff0000u), x[2 * i + 1], acc[r]);
            }
          }
        }
      }
      // the next chunks of this task, or the first of the next one
      if (c0 + 32 * U < chunks) load(task, c0 + 32 * U);
      else if (task + stride < tasks) load(task + stride, 0);
    }
#pragma unroll
    for (int r = 0; r < RW; ++r) acc[r] = warp_sum(acc[r]);
    const int act = second ? v.act2 : a.act, outs = second ? outs2 : outs1, task_at = second ? task - tasks1 : task;
    const float* bias = second ? v.bias2 : a.bias;
    float* out = second ? v.out2 : v.out;
    if (glu_of(act)) {
      if (lane == 0) {
        float g = acc[0], u = acc[RW - 1];
        if (bias) {
          g += bias[task_at];
          u += bias[task_at + outs];
        }
        out[task_at] = (act == ACT_GLU ? siluf_(g) : gelu_tanhf_(g)) * u;
      }
    } else {
#pragma unroll
      for (int r = 0; r < RW; ++r) {
        const int row = task_at * RW + r;
        if (lane == r && row < outs) {
          float y = acc[r];
          if (bias) y += bias[row];
          if (act == ACT_SILU_SIGMOID) y = row < a.act_split ? siluf_(y) : sigmoidf_(y);
          if (act == ACT_SOFTCAP) y = softcapf_(y * a.out_scale, a.softcap);
          out[row] = y;
          if (best_row < 0 || y > best) {   // rows of a lane ascend
            best = y;
            best_row = row;
          }
        }
      }
    }
  }
  if (!v.part_val) return;
  __shared__ float bv[kVecWarps];
  __shared__ int bi[kVecWarps];
  auto better = [](float x, int i, float y, int j) { return i >= 0 && (j < 0 || x > y || (x == y && i < j)); };
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float x = __shfl_xor_sync(0xffffffffu, best, o);
    const int i = __shfl_xor_sync(0xffffffffu, best_row, o);
    if (better(x, i, best, best_row)) {
      best = x;
      best_row = i;
    }
  }
  if (lane == 0) {
    bv[warp] = best;
    bi[warp] = best_row;
  }
  __syncthreads();
  if (tid == 0) {
    for (int w = 1; w < kVecWarps; ++w)
      if (better(bv[w], bi[w], best, best_row)) {
        best = bv[w];
        best_row = bi[w];
      }
    v.part_val[blockIdx.x] = best_row >= 0 ? best : -INFINITY;
    v.part_idx[blockIdx.x] = best_row >= 0 ? best_row : 0x7fffffff;
  }
}

constexpr int kTile = 64, kTileK = 16;
// 64 rows x 64 features per block of 256 threads, 4 x 4 outputs per thread
__global__ void __launch_bounds__(256) linear_f32_kernel(const LinearArgs a, const float* __restrict__ x, int64_t ldx, float* __restrict__ y,
                                                         int64_t ldy) {
  __shared__ float xt[kTileK][kTile + 4], wt[kTileK][kTile + 4];
  const int tid = threadIdx.x, r0 = blockIdx.y * kTile, f0 = blockIdx.x * kTile;
  const int tr = (tid / 16) * 4, tf = (tid % 16) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.w.K; k0 += kTileK) {
    for (int i = tid; i < kTile * kTileK; i += 256) {
      const int row = i / kTileK, k = k0 + i % kTileK;
      xt[i % kTileK][row] = r0 + row < a.rows && k < a.w.K ? x[(int64_t)(r0 + row) * ldx + k] : 0.0f;
      wt[i % kTileK][row] = f0 + row < a.w.M && k < a.w.K ? __bfloat162float(a.w.w[(int64_t)(f0 + row) * a.w.ld + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kTileK; ++k) {
      float xr[4], wr[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        xr[i] = xt[k][tr + i];
        wr[i] = wt[k][tf + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xr[i], wr[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = r0 + tr + i, f = f0 + tf + j;
      if (row >= a.rows || f >= a.w.M) continue;
      float o = acc[i][j];
      if (a.bias) o += a.bias[f];
      if (a.act == ACT_SILU_SIGMOID) o = f < a.act_split ? siluf_(o) : sigmoidf_(o);
      if (a.act == ACT_SOFTCAP) o = softcapf_(o * a.out_scale, a.softcap);
      y[(int64_t)row * ldy + f] = o;
    }
}

}  // namespace

cudaError_t launch_linear_vec(const LinearArgs& a, const VecArgs& v, int sm_count, bool pdl, cudaStream_t st, int* parts) {
  const bool dual = v.w2.w != nullptr;
  const int chunks = (a.w.K + 7) / 8, smem = (dual ? 64 : 32) * chunks;
  if (smem > 200 * 1024 || (dual && (v.w2.K != a.w.K || v.pro != PRO_PRENORM || v.part_val))) return cudaErrorInvalidValue;
  auto outs_of = [](const Bf16Matrix& w, int act) { return is_glu(act) ? w.M / 2 : w.M; };
  const int outs = outs_of(a.w, a.act);
  // two rows per warp unless that leaves SMs without work
  const bool pair = dual || is_glu(a.act) || outs >= sm_count * kVecWarps * 2;
  auto kern = dual ? linear_vec_kernel<2, 4, true> : pair ? linear_vec_kernel<2, 4, false> : linear_vec_kernel<1, 8, false>;
  if (smem > 40 * 1024) {
    // the same limit for every size: launches of other sizes may already be in a captured step
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return e;
  }
  auto tasks_of = [&](int n, int act) { return pair && !is_glu(act) ? (n + 1) / 2 : n; };
  const int tasks = tasks_of(outs, a.act) + (dual ? tasks_of(outs_of(v.w2, v.act2), v.act2) : 0);
  int per_sm = (200 * 1024) / (smem + 1024);
  per_sm = per_sm > 4 ? 4 : per_sm;
  int grid = (tasks + kVecWarps - 1) / kVecWarps;
  if (grid > sm_count * per_sm) grid = sm_count * per_sm;
  if (parts) *parts = grid;
  return launch_kernel(kern, dim3(grid), dim3(kVecThreads), (size_t)smem, st, pdl, a, v);
}

cudaError_t launch_linear_f32(const LinearArgs& a, const float* x, int64_t ldx, float* y, int64_t ldy, cudaStream_t st) {
  if (is_glu(a.act)) return cudaErrorInvalidValue;
  const dim3 grid((a.w.M + kTile - 1) / kTile, (a.rows + kTile - 1) / kTile);
  linear_f32_kernel<<<grid, 256, 0, st>>>(a, x, ldx, y, ldy);
  return cudaGetLastError();
}

}  // namespace emelb
