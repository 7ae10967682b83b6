// Linear attention with a fixed decay per head: S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.  The state
// [dim][vdim] of a (sequence, head) is f32 and stays in HBM between calls; a sequence that starts at position 0 starts
// from zero whatever the memory holds.
#include "common.cuh"
#include "layered.h"

namespace emelb {
namespace {

constexpr int kCols = 32, kGroups = 8;   // value columns per block x row groups of the state

__device__ __forceinline__ float from(float x) { return x; }
__device__ __forceinline__ float from(__nv_bfloat16 x) { return __bfloat162float(x); }

// token by token: grid (heads, column tiles, sequences)
template <class T>
__global__ void __launch_bounds__(kCols * kGroups) linear_attention_rows_kernel(const LinAttnArgs a, const T* __restrict__ x, const Rows rows) {
  extern __shared__ float sm[];
  float* S = sm;                              // [dim][kCols]
  float* ks = S + a.dim * kCols;              // [dim]
  float* qs = ks + a.dim;                     // [dim]
  float* red = qs + a.dim;                    // [kGroups][kCols]
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, col = blockIdx.y * kCols + threadIdx.x, tx = threadIdx.x, ty = threadIdx.y, tid = ty * kCols + tx;
  const int seq = rows.prompt ? rows.seq0 : rows.seq0 + blockIdx.z;
  const int pos = rows.prompt ? rows.pos[0] : rows.pos[blockIdx.z];
  const int first = rows.prompt ? 0 : blockIdx.z, count = rows.prompt ? rows.n : 1;
  const bool live = col < a.vdim;
  float* state = a.state + ((int64_t)seq * a.heads + h) * a.dim * a.vdim;
  for (int i = ty; i < a.dim; i += kGroups) S[i * kCols + tx] = live && pos > 0 ? state[(int64_t)i * a.vdim + col] : 0.0f;
  const float decay = a.decay[h];
  for (int r = first; r < first + count; ++r) {
    const T* row = x + (int64_t)r * a.ldx;
    __syncthreads();
    for (int i = tid; i < a.dim; i += kCols * kGroups) {
      qs[i] = from(row[h * a.dim + i]);
      ks[i] = from(row[(a.heads + h) * a.dim + i]);
    }
    const float v = live ? from(row[2 * a.heads * a.dim + h * a.vdim + col]) : 0.0f;
    __syncthreads();
    float acc = 0.0f;
    for (int i = ty; i < a.dim; i += kGroups) {
      const float s = fmaf(ks[i], v, decay * S[i * kCols + tx]);
      S[i * kCols + tx] = s;
      acc = fmaf(qs[i], s, acc);
    }
    red[ty * kCols + tx] = acc;
    __syncthreads();
    if (ty == 0 && live) {
      float o = 0.0f;
#pragma unroll
      for (int g = 0; g < kGroups; ++g) o += red[g * kCols + tx];
      a.out[((int64_t)r * a.heads + h) * a.vdim + col] = o;
    }
  }
  if (live)
    for (int i = ty; i < a.dim; i += kGroups) state[(int64_t)i * a.vdim + col] = S[i * kCols + tx];
}

}  // namespace

template <class T>
cudaError_t launch_linear_attention_rows(const LinAttnArgs& a, const T* x, const Rows& rows, cudaStream_t st) {
  const size_t smem = 4 * ((size_t)a.dim * kCols + 2 * a.dim + kGroups * kCols);
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(linear_attention_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  linear_attention_rows_kernel<T><<<dim3(a.heads, (a.vdim + kCols - 1) / kCols, rows.prompt ? 1 : rows.n), dim3(kCols, kGroups), smem, st>>>(a, x, rows);
  return cudaGetLastError();
}
template cudaError_t launch_linear_attention_rows<float>(const LinAttnArgs&, const float*, const Rows&, cudaStream_t);
template cudaError_t launch_linear_attention_rows<__nv_bfloat16>(const LinAttnArgs&, const __nv_bfloat16*, const Rows&, cudaStream_t);

bool linear_attention_prompt_supported(const LinAttnArgs&) { return false; }
cudaError_t launch_linear_attention_prompt(const LinAttnArgs&, const __nv_bfloat16*, const Rows&, cudaStream_t) { return cudaErrorInvalidValue; }

}  // namespace emelb
