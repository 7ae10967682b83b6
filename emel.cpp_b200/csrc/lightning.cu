// Linear attention with a fixed decay per head: S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.  The state
// [dim][vdim] of a (sequence, head) is f32 and stays in HBM between calls; a sequence that starts at position 0 starts
// from zero whatever the memory holds.
#include "common.cuh"
#include "layered.h"
#include "mma_bf16.cuh"

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

// ---- prompts on the tensor cores (mma.sync bf16, f32 accumulators), chunk by chunk.  With the state S before a chunk of
// n tokens:
//   o_i  = decay^(i+1) S^T q_i + sum_(j<=i) decay^(i-j) (q_i . k_j) v_j
//   S'   = decay^n S + sum_j decay^(n-1-j) k_j v_j^T
// q, k and v are bf16; every f32 factor that meets them (the state, the decayed scores, the decayed values) is fed as
// two bf16 operands, high part and remainder, so the recurrence keeps f32 accuracy.
// Long prompts are cut into segments of whole chunks that run side by side: a first launch (STATES) leaves what each
// segment but the last adds to the state in `local`, the second starts every segment from the sum of those before it.
// One block = one head x kVS value columns, four warps: 16 query rows each for the outputs, every fourth 16-row tile of
// the state, which lives in accumulator fragments between the chunks.
constexpr int kChunk = 64, kVS = 32, kMmaThreads = 128;

template <int D>
struct ChunkSmem {
  static constexpr int kRow = D + 8, kVRow = kVS + 8;
  __nv_bfloat16 q[2][kChunk][kRow], k[2][kChunk][kRow], v[2][kChunk][kVRow];
  __nv_bfloat16 s_hi[D][kVRow], s_lo[D][kVRow];
  float pw[kChunk + 1];
};

// local: [segment][head][D][vdim]; with several segments its last entry holds the state the prompt starts from, since
// the sequence's own is overwritten while other segments may not have started
template <int D, bool STATES>
__global__ void __launch_bounds__(kMmaThreads) linear_attention_prompt_kernel(const LinAttnArgs a, const __nv_bfloat16* __restrict__ x, const Rows rows,
                                                                              const int segment, const int segments) {
  extern __shared__ __align__(16) unsigned char raw[];
  using Smem = ChunkSmem<D>;
  Smem& sm = *reinterpret_cast<Smem*>(raw);
  constexpr int KS = D / 16, MT = (KS + 3) / 4, NT = kVS / 8;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int h = blockIdx.x, v0 = blockIdx.y * kVS;
  const float decay = a.decay[h];
  float* state = a.state + ((int64_t)rows.seq0 * a.heads + h) * D * a.vdim;
  auto local = [&](int seg) { return a.local + ((int64_t)seg * a.heads + h) * D * a.vdim; };
  const int seg = blockIdx.z, row_begin = seg * segment, row_end = min(rows.n, row_begin + segment);
  const __nv_bfloat16 *xq = x + h * D, *xk = x + (a.heads + h) * D, *xv = x + 2 * a.heads * D + h * a.vdim + v0;

  auto issue = [&](int c0, int buf) {
    for (int i = tid; i < kChunk * (D / 8); i += kMmaThreads) {
      const int r = i / (D / 8), c = i % (D / 8) * 8;
      const bool live = c0 + r < row_end;
      const int64_t at = (int64_t)(live ? c0 + r : 0) * a.ldx + c;
      if (!STATES) cp16_zfill(&sm.q[buf][r][c], xq + at, live);
      cp16_zfill(&sm.k[buf][r][c], xk + at, live);
    }
    for (int i = tid; i < kChunk * (kVS / 8); i += kMmaThreads) {
      const int r = i / (kVS / 8), c = i % (kVS / 8) * 8;
      const bool live = c0 + r < row_end && v0 + c < a.vdim;
      cp16_zfill(&sm.v[buf][r][c], live ? xv + (int64_t)(c0 + r) * a.ldx + c : xq, live);
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  issue(row_begin, 0);
  for (int i = tid; i <= kChunk; i += kMmaThreads) sm.pw[i] = powf(decay, (float)i);

  // state rows 16 (warp + 4 mt) + g (+8), columns 8 nt + 2t (+1)
  float S[MT][NT][4];
  const bool carried = rows.pos[0] > 0;
  const float across = powf(decay, (float)segment);   // one whole segment's decay
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = 16 * (warp + 4 * mt) + g + 8 * (e >> 1), c = 8 * nt + 2 * t + (e & 1);
        const bool mine = r < D && v0 + c < a.vdim;
        const int64_t at = (int64_t)r * a.vdim + v0 + c;
        float v = 0.0f;
        if (STATES) {
          if (mine && seg == 0) {
            v = carried ? state[at] : 0.0f;
            local(segments - 1)[at] = v;
          }
        } else if (mine) {
          if (seg > 0) {
            v = local(0)[at];   // the first segment's includes the state the prompt starts from
            for (int p = 1; p < seg; ++p) v = fmaf(across, v, local(p)[at]);
          } else if (segments > 1) {
            v = local(segments - 1)[at];
          } else if (carried) {
            v = state[at];
          }
        }
        S[mt][nt][e] = v;
      }
  auto publish = [&]() {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      if (warp + 4 * mt >= KS) continue;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t hi, lo;
          split2(S[mt][nt][2 * half], S[mt][nt][2 * half + 1], hi, lo);
          const int r = 16 * (warp + 4 * mt) + g + 8 * half, c = 8 * nt + 2 * t;
          *reinterpret_cast<uint32_t*>(&sm.s_hi[r][c]) = hi;
          *reinterpret_cast<uint32_t*>(&sm.s_lo[r][c]) = lo;
        }
    }
  };
  if (!STATES) publish();

  int buf = 0;
  for (int c0 = row_begin; c0 < row_end; c0 += kChunk, buf ^= 1) {
    const int n = min(kChunk, row_end - c0);
    if (c0 + kChunk < row_end) {
      issue(c0 + kChunk, buf ^ 1);
      asm volatile("cp.async.wait_group 1;\n" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    }
    __syncthreads();
    const int r0 = 16 * warp;   // this warp's query rows
    if (!STATES && r0 < n) {
      float s[kChunk / 8][4] = {}, o[NT][4] = {};
      const int ktiles = warp + 1;   // keys up to this warp's last row, 16 at a time
#pragma unroll
      for (int kk = 0; kk < KS; ++kk) {
        uint32_t q[4];
        ldsm(q, &sm.q[buf][r0 + (lane & 15)][16 * kk + (lane >> 4) * 8]);
#pragma unroll
        for (int kt = 0; kt < kChunk / 16; ++kt) {
          if (kt >= ktiles) break;
          uint32_t b[4];
          ldsm(b, &sm.k[buf][16 * kt + (lane & 7) + (lane >> 4) * 8][16 * kk + ((lane >> 3) & 1) * 8]);
          mma_bf16_16816(s[2 * kt], q, b[0], b[1]);
          mma_bf16_16816(s[2 * kt + 1], q, b[2], b[3]);
        }
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          uint32_t b[4];
          ldsm_trans(b, &sm.s_hi[16 * kk + (lane & 15)][16 * np + (lane >> 4) * 8]);
          mma_bf16_16816(o[2 * np], q, b[0], b[1]);
          mma_bf16_16816(o[2 * np + 1], q, b[2], b[3]);
          ldsm_trans(b, &sm.s_lo[16 * kk + (lane & 15)][16 * np + (lane >> 4) * 8]);
          mma_bf16_16816(o[2 * np], q, b[0], b[1]);
          mma_bf16_16816(o[2 * np + 1], q, b[2], b[3]);
        }
      }
      const float d0 = sm.pw[r0 + g + 1], d1 = sm.pw[r0 + g + 9];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        o[nt][0] *= d0;
        o[nt][1] *= d0;
        o[nt][2] *= d1;
        o[nt][3] *= d1;
      }
#pragma unroll
      for (int kt = 0; kt < kChunk / 16; ++kt) {
        if (kt >= ktiles) break;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int i = r0 + g + 8 * half, j = 16 * kt + 8 * part + 2 * t;
            const float* p = s[2 * kt + part];
            const float p0 = j <= i ? p[2 * half] * sm.pw[i - j] : 0.0f, p1 = j + 1 <= i ? p[2 * half + 1] * sm.pw[i - j - 1] : 0.0f;
            split2(p0, p1, hi[2 * part + half], lo[2 * part + half]);
          }
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          uint32_t b[4];
          ldsm_trans(b, &sm.v[buf][16 * kt + (lane & 15)][16 * np + (lane >> 4) * 8]);
          mma_bf16_16816(o[2 * np], hi, b[0], b[1]);
          mma_bf16_16816(o[2 * np], lo, b[0], b[1]);
          mma_bf16_16816(o[2 * np + 1], hi, b[2], b[3]);
          mma_bf16_16816(o[2 * np + 1], lo, b[2], b[3]);
        }
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = c0 + r0 + g + 8 * half;
        if (i >= row_end) continue;
        float* out = a.out + ((int64_t)i * a.heads + h) * a.vdim + v0;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const int c = 8 * nt + 2 * t;
          if (v0 + c < a.vdim) *reinterpret_cast<float2*>(out + c) = make_float2(o[nt][2 * half], o[nt][2 * half + 1]);
        }
      }
    }
    // the state after this chunk
    const float dn = sm.pw[n];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[mt][nt][e] *= dn;
#pragma unroll
    for (int kt = 0; kt < kChunk / 16; ++kt) {
      if (16 * kt >= n) break;
      // decayed values of these 16 tokens; the rows past the end are zero
      uint32_t hi[NT][2], lo[NT][2];
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        uint32_t b[4];
        ldsm_trans(b, &sm.v[buf][16 * kt + (lane & 15)][16 * np + (lane >> 4) * 8]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int j = 16 * kt + 8 * (i & 1) + 2 * t;
          const float2 v = unpack2(b[i]);
          const float w0 = j < n ? sm.pw[n - 1 - j] : 0.0f, w1 = j + 1 < n ? sm.pw[n - 2 - j] : 0.0f;
          split2(v.x * w0, v.y * w1, hi[2 * np + (i >> 1)][i & 1], lo[2 * np + (i >> 1)][i & 1]);
        }
      }
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        if (warp + 4 * mt >= KS) continue;
        uint32_t k[4];
        ldsm_trans(k, &sm.k[buf][16 * kt + (lane & 7) + (lane >> 4) * 8][16 * (warp + 4 * mt) + ((lane >> 3) & 1) * 8]);
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          mma_bf16_16816(S[mt][nt], k, hi[nt][0], hi[nt][1]);
          mma_bf16_16816(S[mt][nt], k, lo[nt][0], lo[nt][1]);
        }
      }
    }
    __syncthreads();   // every warp is done with this chunk and with the old state
    if (!STATES) publish();
  }
  if (!STATES && seg != segments - 1) return;
  float* dst = STATES ? local(seg) : state;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = 16 * (warp + 4 * mt) + g + 8 * (e >> 1), c = 8 * nt + 2 * t + (e & 1);
        if (r < D && v0 + c < a.vdim) dst[(int64_t)r * a.vdim + v0 + c] = S[mt][nt][e];
      }
}

template <int D>
cudaError_t launch_prompt(const LinAttnArgs& a, const __nv_bfloat16* x, const Rows& rows, int sm_count, cudaStream_t st, int* launches) {
  const int smem = (int)sizeof(ChunkSmem<D>);
  cudaError_t e = cudaFuncSetAttribute(linear_attention_prompt_kernel<D, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(linear_attention_prompt_kernel<D, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  const int tiles = (a.vdim + kVS - 1) / kVS;
  // segments of at least 256 tokens while two blocks per SM have room for them
  int segments = 2 * sm_count / (a.heads * tiles);
  if (segments > kLinAttnMaxSegments) segments = kLinAttnMaxSegments;
  if (segments > rows.n / 256) segments = rows.n / 256;
  if (segments < 2 || !a.local) segments = 1;
  const int chunks = (rows.n + kChunk - 1) / kChunk, segment = (chunks + segments - 1) / segments * kChunk;
  segments = (rows.n + segment - 1) / segment;
  if (segments > 1) {
    linear_attention_prompt_kernel<D, true><<<dim3(a.heads, tiles, segments - 1), kMmaThreads, smem, st>>>(a, x, rows, segment, segments);
    *launches += 1;
  }
  linear_attention_prompt_kernel<D, false><<<dim3(a.heads, tiles, segments), kMmaThreads, smem, st>>>(a, x, rows, segment, segments);
  *launches += 1;
  return cudaGetLastError();
}

}  // namespace

bool linear_attention_prompt_supported(const LinAttnArgs& a) {
  return a.dim % 16 == 0 && a.dim <= 128 && a.vdim % 8 == 0 && a.ldx % 8 == 0;
}

cudaError_t launch_linear_attention_prompt(const LinAttnArgs& a, const __nv_bfloat16* x, const Rows& rows, int sm_count, cudaStream_t st,
                                           int* launches) {
  switch (a.dim / 16) {
    case 1: return launch_prompt<16>(a, x, rows, sm_count, st, launches);
    case 2: return launch_prompt<32>(a, x, rows, sm_count, st, launches);
    case 3: return launch_prompt<48>(a, x, rows, sm_count, st, launches);
    case 4: return launch_prompt<64>(a, x, rows, sm_count, st, launches);
    case 5: return launch_prompt<80>(a, x, rows, sm_count, st, launches);
    case 6: return launch_prompt<96>(a, x, rows, sm_count, st, launches);
    case 7: return launch_prompt<112>(a, x, rows, sm_count, st, launches);
    case 8: return launch_prompt<128>(a, x, rows, sm_count, st, launches);
    default: return cudaErrorInvalidValue;
  }
}

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

}  // namespace emelb
