// y {rows, M} = act(x {rows, K} W {M, K}^T + bias) with bf16 operands on the Blackwell tensor cores: tcgen05.mma
// kind::f16, f32 accumulators in TMEM, operands brought by TMA in the 128-byte swizzled K-major layout.
//
// The weights are the M operand (128 rows = TMEM lanes), BN rows of x the N operand, so few rows cost a narrow tile.
// One output tile per CTA, 6 warps: warps 0-3 read the accumulators back (one TMEM lane quarter each), warp 4 issues
// the TMA copies, warp 5 owns the TMEM allocation and issues the MMAs.  GLU tiles hold a gate tile and the up tile of
// the same outputs side by side in TMEM and store silu(gate) * up.
// Every wait is bounded; on a timeout the CTA raises the status word, lets its copies land and frees its TMEM.
#include <cuda.h>
#include <cudaTypedefs.h>
#include <cuda_runtime.h>

#include "act.cuh"
#include "common.cuh"
#include "layered.h"

namespace emelb {
namespace {

constexpr int kThreads = 192, kTmaWarp = 4, kMmaWarp = 5;
constexpr int kBM = kGemmWeightBox, kBK = 64;
constexpr int kWeightTile = kBM * kBK * 2;
constexpr int kWaitSpins = 1 << 22;
constexpr uint32_t kSuspendHintNs = 10000;
constexpr unsigned long long kWaitNs = 2000000000ull;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void mbar_init(uint64_t* bar, int count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count) : "memory");
}
__device__ __forceinline__ void mbar_arrive_expect_tx(uint64_t* bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes) : "memory");
}
__device__ __forceinline__ bool mbar_try_wait(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2, %3;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity), "r"(kSuspendHintNs)
      : "memory");
  return ok != 0;
}
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag) {
  unsigned long long t0 = 0;
  for (int spins = 0; spins < kWaitSpins; ++spins) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((spins & 15) == 15) {
      if (*abort_flag) return false;
      unsigned long long now;
      asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(now));
      if (t0 == 0) t0 = now;
      else if (now - t0 > kWaitNs) break;
    }
  }
  *abort_flag = 1;
  return false;
}
__device__ __forceinline__ void tma_load(void* dst, const TmaMap* map, int x, int y, uint64_t* bar) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(smem_u32(dst)),
               "l"(map), "r"(x), "r"(y), "r"(smem_u32(bar))
               : "memory");
}
// K-major operand in 8-row x 128-byte swizzled atoms, 1024 bytes apart (descriptor version 1, swizzle mode 2)
__device__ __forceinline__ uint64_t operand_desc(uint32_t saddr) {
  return (uint64_t)((saddr >> 4) & 0x3fffu) | (uint64_t)1 << 16 | (uint64_t)(1024 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)2 << 61;
}
// D = f32, A = B = bf16, both K-major, M = 128
template <int BN>
constexpr uint32_t kInstrDesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kBM >> 4) << 24);
__device__ __forceinline__ void mma_bf16(uint32_t tmem_d, uint64_t da, uint64_t db, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(tmem_d), "l"(da), "l"(db), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void mma_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void tmem_ld(uint32_t taddr, uint32_t (&v)[16]) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 "
               "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
               : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
                 "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
               : "r"(taddr)
               : "memory");
}
__device__ __forceinline__ void tmem_ld(uint32_t taddr, uint32_t (&v)[32]) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x32.b32 "
               "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
               "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
               : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
                 "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]),
                 "=r"(v[16]), "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]),
                 "=r"(v[24]), "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
               : "r"(taddr)
               : "memory");
}

struct GemmParams {
  int M, K, rows;          // M: outputs (half of the stored rows for GLU)
  const float* bias;
  int act, act_split;
  float* y;
  __nv_bfloat16* yb;
  int64_t ldy;
  int* status;
  float out_scale, softcap;
  int tail;                // first feature stored as f32 at tail_y
  float* tail_y;
  int64_t tail_ld;
};

template <int BN, bool GLU>
struct Tile {
  static constexpr int kStageBytes = (GLU ? 2 : 1) * kWeightTile + BN * kBK * 2;
  static constexpr int kStages = kStageBytes > 40 * 1024 ? 2 : BN == 128 ? 3 : 4;   // two CTAs per SM: one computes while the other stores
  static constexpr int kTmemCols = (GLU ? 2 : 1) * BN < 32 ? 32 : (GLU ? 2 : 1) * BN;
  static constexpr int kBox = BN >= 128 ? 128 : kGemmTokenBox;   // rows per TMA copy of x
  static constexpr int kSmem = kStages * kStageBytes + 1024 + 256;
};

template <int BN, bool GLU>
__global__ void __launch_bounds__(kThreads) gemm_bf16_kernel(const __grid_constant__ TmaMap wmap, const __grid_constant__ TmaMap xmap,
                                                             const GemmParams p) {
  using T = Tile<BN, GLU>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + T::kStages * T::kStageBytes);
  uint64_t* empty = full + T::kStages;
  uint64_t* done = empty + T::kStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * BN, f0 = blockIdx.y * kBM;
  const int nk = (p.K + kBK - 1) / kBK;

  if (threadIdx.x == 0) {
    for (int s = 0; s < T::kStages; ++s) {
      mbar_init(full + s, 1);
      mbar_init(empty + s, 1);
    }
    mbar_init(done, 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == kMmaWarp) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(T::kTmemCols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = *tmem_slot;

  if (warp == kTmaWarp && lane == 0) {
    int issued = 0;
    for (int i = 0; i < nk; ++i) {
      const int s = i % T::kStages;
      if (i >= T::kStages && !mbar_wait(empty + s, ((i / T::kStages) - 1) & 1, abort_flag)) break;
      uint8_t* st = smem + s * T::kStageBytes;
      mbar_arrive_expect_tx(full + s, T::kStageBytes);
      tma_load(st, &wmap, i * kBK, f0, full + s);
      if (GLU) tma_load(st + kWeightTile, &wmap, i * kBK, p.M + f0, full + s);
      uint8_t* xt = st + (GLU ? 2 : 1) * kWeightTile;
#pragma unroll
      for (int b = 0; b < BN / T::kBox; ++b) tma_load(xt + b * T::kBox * kBK * 2, &xmap, i * kBK, t0 + b * T::kBox, full + s);
      issued = i + 1;
    }
    // after a timeout: let the copies in flight land before the memory goes away
    if (*abort_flag)
      for (int i = issued > T::kStages ? issued - T::kStages : 0; i < issued; ++i)
        for (int spin = 0; spin < 1 << 16 && !mbar_try_wait(full + i % T::kStages, (i / T::kStages) & 1); ++spin) {}
  } else if (warp == kMmaWarp && lane == 0) {
    for (int i = 0; i < nk; ++i) {
      const int s = i % T::kStages;
      if (!mbar_wait(full + s, (i / T::kStages) & 1, abort_flag)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t st = smem_u32(smem + s * T::kStageBytes);
      const uint32_t xt = st + (GLU ? 2 : 1) * kWeightTile;
#pragma unroll
      for (int k = 0; k < kBK / 16; ++k) {
        const uint64_t db = operand_desc(xt + 32 * k);
        mma_bf16(tmem, operand_desc(st + 32 * k), db, kInstrDesc<BN>, i > 0 || k > 0);
        if (GLU) mma_bf16(tmem + BN, operand_desc(st + kWeightTile + 32 * k), db, kInstrDesc<BN>, i > 0 || k > 0);
      }
      mma_commit(empty + s);
    }
    mma_commit(done);
    if (*abort_flag)   // after a timeout: let the MMAs in flight end before the accumulators are freed
      for (int spin = 0; spin < 1 << 16 && !mbar_try_wait(done, 0); ++spin) {}
  }
  __syncwarp();
  if (warp < 4) {
    if (mbar_wait(done, 0, abort_flag) && !*abort_flag) {
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      __syncwarp();
      const int f = f0 + warp * 32 + lane;
      const bool live = f < p.M;
      const float b0 = live && p.bias ? p.bias[f] : 0.0f, b1 = GLU && live && p.bias ? p.bias[p.M + f] : 0.0f;
      const uint32_t lane_base = tmem + ((uint32_t)(warp * 32) << 16);
      const bool sigm = p.act == ACT_SILU_SIGMOID, gelu = p.act == ACT_GLU_GELU, cap = p.act == ACT_SOFTCAP, tail = f >= p.tail;
      // bf16 outputs turn in shared memory (the stages are free: every copy has landed and been used), 32 features x kCh rows of
      // a warp at a time, and leave as 16-byte stores
      constexpr int kCh = BN < 32 ? BN : 32, kTileLd = 40;
      __nv_bfloat16* tile = reinterpret_cast<__nv_bfloat16*>(smem) + warp * 32 * kTileLd;
      const int f_end = min(p.M, p.tail), fw = f0 + warp * 32;
      for (int c = 0; c < BN && t0 + c < p.rows; c += kCh) {
        uint32_t v[kCh], u[GLU ? kCh : 1];
        tmem_ld(lane_base + c, v);
        if constexpr (GLU) tmem_ld(lane_base + BN + c, u);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        float o[kCh];
#pragma unroll
        for (int j = 0; j < kCh; ++j) {
          o[j] = __uint_as_float(v[j]) + b0;
          if constexpr (GLU) {
            o[j] = (gelu ? gelu_tanhf_(o[j]) : siluf_(o[j])) * (__uint_as_float(u[j]) + b1);
          } else if (sigm) {
            const float sg = sigmoidf_(o[j]);
            o[j] = f < p.act_split ? o[j] * sg : sg;
          } else if (cap) {
            o[j] = softcapf_(o[j] * p.out_scale, p.softcap);
          }
        }
        if (live && (tail || !p.yb)) {
          float* y = tail ? p.tail_y + f - p.tail : p.y + f;
          const int64_t ld = tail ? p.tail_ld : p.ldy;
#pragma unroll
          for (int j = 0; j < kCh; ++j)
            if (t0 + c + j < p.rows) y[(int64_t)(t0 + c + j) * ld] = o[j];
        }
        if (!p.yb) continue;
        __syncwarp();
#pragma unroll
        for (int j = 0; j < kCh; ++j) tile[j * kTileLd + lane] = __float2bfloat16_rn(o[j]);
        __syncwarp();
#pragma unroll
        for (int i = lane; i < 4 * kCh; i += 32) {
          const int j = i / 4, q = 8 * (i % 4), n = f_end - fw - q;   // n features of this piece are stored
          if (t0 + c + j >= p.rows || n <= 0) continue;
          const __nv_bfloat16* src = tile + j * kTileLd + q;
          __nv_bfloat16* dst = p.yb + (int64_t)(t0 + c + j) * p.ldy + fw + q;
          if (n >= 8) {
            *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
          } else {
            for (int e = 0; e < n; ++e) dst[e] = src[e];
          }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (threadIdx.x == 0 && *abort_flag && p.status) atomicExch(p.status, 1);
  if (warp == kMmaWarp) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(T::kTmemCols) : "memory");
  }
}

template <int BN, bool GLU>
cudaError_t launch_tile(const TmaMap& wmap, const TmaMap& xmap, const GemmParams& p, cudaStream_t st) {
  using T = Tile<BN, GLU>;
  const cudaError_t e = cudaFuncSetAttribute(gemm_bf16_kernel<BN, GLU>, cudaFuncAttributeMaxDynamicSharedMemorySize, T::kSmem);
  if (e != cudaSuccess) return e;
  gemm_bf16_kernel<BN, GLU><<<dim3((p.rows + BN - 1) / BN, (p.M + kBM - 1) / kBM), kThreads, T::kSmem, st>>>(wmap, xmap, p);
  return cudaGetLastError();
}

}  // namespace

bool encode_bf16_map(TmaMap* map, const __nv_bfloat16* base, int64_t rows, int64_t k, int64_t ld, int box_rows) {
  static_assert(sizeof(CUtensorMap) == sizeof(TmaMap), "tensor map size");
  if (reinterpret_cast<uintptr_t>(base) % 16 != 0 || ld % 8 != 0 || rows < 1 || k < 1) return false;
  static PFN_cuTensorMapEncodeTiled_v12000 encode = nullptr;
  if (!encode) {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &fn, 12000, cudaEnableDefault, &q) != cudaSuccess || !fn) {
      cudaGetLastError();
      return false;
    }
    encode = reinterpret_cast<PFN_cuTensorMapEncodeTiled_v12000>(fn);
  }
  const cuuint64_t dims[2] = {(cuuint64_t)k, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
  const cuuint32_t box[2] = {(cuuint32_t)kBK, (cuuint32_t)box_rows}, estr[2] = {1, 1};
  return encode(reinterpret_cast<CUtensorMap*>(map), CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<__nv_bfloat16*>(base), dims, strides, box, estr,
                CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

cudaError_t launch_gemm_bf16(const LinearArgs& a, const TmaMap& wmap, const XMaps& x, float* y, __nv_bfloat16* yb, int64_t ldy, int* status,
                             cudaStream_t st) {
  if (yb && (ldy % 8 != 0 || reinterpret_cast<uintptr_t>(yb) % 16 != 0)) return cudaErrorInvalidValue;
  const bool glu = is_glu(a.act);
  GemmParams p{glu ? a.w.M / 2 : a.w.M, a.w.K, a.rows, a.bias, a.act, a.act_split, y, yb, ldy, status,
               a.out_scale, a.softcap, a.tail, a.tail_y, a.tail_ld};
  const int R = a.rows;
  if (glu) {
    if (R <= 16) return launch_tile<16, true>(wmap, x.narrow, p, st);
    if (R <= 64) return launch_tile<64, true>(wmap, x.narrow, p, st);
    return launch_tile<128, true>(wmap, x.wide, p, st);
  }
  if (R <= 16) return launch_tile<16, false>(wmap, x.narrow, p, st);
  if (R <= 64) return launch_tile<64, false>(wmap, x.narrow, p, st);
  // 256-row tiles once there are more of them than SMs
  if (((p.M + kBM - 1) / kBM) * ((R + 255) / 256) >= 180) return launch_tile<256, false>(wmap, x.wide, p, st);
  return launch_tile<128, false>(wmap, x.wide, p, st);
}

}  // namespace emelb
