// Layered decoder sessions (include/emelb_llama.h): the kernels' launch interface and the model object a session
// drives.  Activations are row-major here, one row per token: element e of row r at x[r * ld + e].
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../../include/emelb_llama.h"
#include "kernels.h"

namespace emelb {

// Rows of one launch.  prompt: row r is token pos[0] + r of sequence seq0; otherwise row r is token pos[r] of
// sequence seq0 + r.  Positions live in device memory so that captured steps can be replayed.
struct Rows {
  int n;
  bool prompt;
  int seq0;
  const int* pos;
};

enum Act : int { ACT_NONE = 0, ACT_SILU_SIGMOID = 1, ACT_GLU = 2 };

// ---- linear.cu: products with bf16 weights
// y {rows, M} = act(x W^T + bias).  ACT_SILU_SIGMOID: silu on features below act_split, sigmoid on the others.
// ACT_GLU: W holds M gate rows, then M up rows (bias likewise); y = silu(gate) * up.
struct Bf16Matrix {
  const __nv_bfloat16* w = nullptr;
  int64_t ld = 0;    // elements between rows, a multiple of 8; zeros between K and ld
  int M = 0, K = 0;
};
struct LinearArgs {
  Bf16Matrix w;      // M counts the stored rows (2 x outputs for ACT_GLU)
  const float* bias; // null: none
  int act, act_split;
  int rows;
};
// what the one-row kernel does to its input before the product, in every block
enum Prologue : int {
  PRO_PLAIN = 0,       // x
  PRO_EMBED = 1,       // row *token of the bf16 table, also written to x_out
  PRO_RESIDUAL = 2,    // x + layer_norm(y) * norm_w, also written to x_out
  PRO_RESIDUAL_NORM = 3,  // layer_norm(that) * norm2_w
  PRO_RMS_GATE = 4,    // rms_norm(x) * norm_w * gate
};
struct VecArgs {
  int pro;
  const float* x;
  const float* y;          // PRO_RESIDUAL*
  const float* norm_w;
  const float* norm2_w;
  const float* gate;
  float eps;
  float* x_out;
  const __nv_bfloat16* table;
  int64_t table_ld;
  const int* token;
  float* out;
  float* part_val;         // optional: each block's highest output and the lowest row that has it (kMaxArgmaxParts)
  int* part_idx;
};
// parts (optional): blocks launched
cudaError_t launch_linear_vec(const LinearArgs& a, const VecArgs& v, int sm_count, bool pdl, cudaStream_t st, int* parts = nullptr);
// f32 operands on the CUDA cores
cudaError_t launch_linear_f32(const LinearArgs& a, const float* x, int64_t ldx, float* y, int64_t ldy, cudaStream_t st);

// ---- gemm_bf16.cu: bf16 operands on the tensor cores (tcgen05, TMA); y f32 or bf16
struct TmaMap { alignas(64) unsigned char bytes[128]; };
// {rows, K} row-major bf16 matrix as K-slabs of 64 elements x box_rows rows
bool encode_bf16_map(TmaMap* map, const __nv_bfloat16* base, int64_t rows, int64_t k, int64_t ld, int box_rows);
constexpr int kGemmWeightBox = 128, kGemmTokenBox = 16;
struct XMaps { TmaMap narrow, wide; };   // the activations as boxes of kGemmTokenBox and of 128 rows
cudaError_t launch_gemm_bf16(const LinearArgs& a, const TmaMap& wmap, const XMaps& x, float* y, __nv_bfloat16* yb, int64_t ldy,
                             int* status, cudaStream_t st);

// ---- mixer_ops.cu: row kernels between the products.  T = operand type of the following product (float or bf16)
template <class T>
cudaError_t launch_embed_rows_bf16(const __nv_bfloat16* table, int64_t ld, const int* tokens, int rows, int width, float* x, T* xb,
                                   int64_t ldb, cudaStream_t st);
// x += layer_norm(y) * w; xb = T(x); keep (optional) = a copy of x
template <class T>
cudaError_t launch_residual_norm(float* x, const float* y, const float* w, float eps, int rows, int width, T* xb, int64_t ldb, float* keep,
                                 cudaStream_t st);
// out row r = T(layer_norm(x row index[r]) * w)   (index null: r)
template <class T>
cudaError_t launch_norm_rows(const float* x, const int* index, const float* w, float eps, int rows, int width, T* out, int64_t ldo,
                             cudaStream_t st);
template <class T>
cudaError_t launch_rms_gate(const float* o, const float* w, const T* gate, int64_t ldg, float eps, int rows, int width, T* out, int64_t ldo,
                            cudaStream_t st);
// gate|up {rows, 2 ff} -> silu(gate) * up
cudaError_t launch_glu_rows(const float* gu, int rows, int ff, float* out, int64_t ldo, cudaStream_t st);

struct AttnInArgs {
  const float* proj;       // {rows, channels}: q | k | v, or q alone
  int channels;
  const float* conv;       // [taps][channels]; null: no convolution
  int taps;
  float* conv_state;       // [sequence][taps - 1][channels]
  const float *norm_q, *norm_k;   // null: no norm
  int norm_v;
  float eps;
  int heads, kv_heads, dim, vdim, dim_pad, vdim_pad;
  int own_kv;
  const float *rope_cos, *rope_sin;   // [position][rope_dim / 2]
  int rope_dim;
  void* q;                 // T {rows, heads, dim_pad}
  void *k, *v;             // T caches [sequence][kv head][capacity][pad]
  int64_t capacity;
};
template <class T>
cudaError_t launch_attn_in(const AttnInArgs& a, const Rows& rows, cudaStream_t st);
// the last taps - 1 projected rows become the sequence's state (prompts; single rows do it in launch_attn_in)
cudaError_t launch_conv_state(const AttnInArgs& a, const Rows& rows, cudaStream_t st);

// ---- mixed_attention.cu
struct MixAttnArgs {
  const void* q;           // T {rows, heads, dim_pad}
  const void *k, *v;       // T caches
  int64_t capacity;
  int heads, kv_heads, dim_pad, vdim, vdim_pad;
  float scale;
  int window, keep_first;
  const float* talk;       // [heads][heads]; null: none
  float* scores;           // scratch
  uint64_t scores_floats;
  float* stats;            // scratch {max, sum} pairs
  uint64_t stats_floats;
  float* part;             // scratch partial outputs
  uint64_t part_floats;
  int max_visible;         // most keys a query of this session can see
};
constexpr int kMixAttnMaxSplits = 32;
int mix_attn_splits(const MixAttnArgs& a, int sm_count);
// out {rows, heads * vdim} of type TO
template <class T, class TO>
cudaError_t launch_mix_attention_rows(const MixAttnArgs& a, const Rows& rows, TO* out, int64_t ldo, int sm_count, cudaStream_t st, int* launches);
// prompts on the tensor cores; pos0 = host copy of rows.pos[0]
bool mix_attention_prompt_supported(const MixAttnArgs& a);
cudaError_t launch_mix_attention_prompt(const MixAttnArgs& a, const Rows& rows, int pos0, __nv_bfloat16* out, int64_t ldo, cudaStream_t st, int* launches);

// ---- lightning.cu: S = decay S + k v^T, o = S^T q
struct LinAttnArgs {
  int64_t ldx;             // q | k | v | gate rows
  int heads, dim, vdim;
  const float* decay;      // device, [heads]
  float* state;            // [sequence][heads][dim][vdim]
  float* out;              // {rows, heads * vdim}
  float* local;            // scratch of kLinAttnMaxSegments states (null: prompts run as one segment)
};
constexpr int kLinAttnMaxSegments = 8;
template <class T>
cudaError_t launch_linear_attention_rows(const LinAttnArgs& a, const T* x, const Rows& rows, cudaStream_t st);
bool linear_attention_prompt_supported(const LinAttnArgs& a);
cudaError_t launch_linear_attention_prompt(const LinAttnArgs& a, const __nv_bfloat16* x, const Rows& rows, int sm_count, cudaStream_t st,
                                           int* launches);

// ---- layered.cu: the model object
struct Layered;
struct LayeredRun {
  cudaStream_t st;
  int launches = 0;
  bool ok = true;
};
uint32_t layered_check(const emelb_llama_config& cfg, const emelb_layer_config* layers);
Layered* layered_create(emelb_ctx* c, const emelb_llama_config& cfg, const emelb_layer_config* layers, bool f32);
void layered_destroy(Layered* m);
uint32_t layered_bind(Layered* m, int layer, int role, const emelb_view* t);
bool layered_bound(const Layered* m);
bool layered_set_sequences(Layered* m, int n_seq);   // sizes and clears the sequences' caches and state
bool layered_reserve_rows(Layered* m, int rows);
int layered_row_capacity(const Layered* m);
void layered_set_trace(Layered* m, float* out, int max_tokens);
// one token of sequence seq; state = {token, position, ...} on the device; logits null: none
// argmax_parts (optional): with logits, the context's argmax candidates are written too; their count
void layered_step(Layered* m, LayeredRun& r, int seq, const int* state, float* logits, int* argmax_parts = nullptr);
// rows through every layer; pos0: host copy of the first position (prompts)
void layered_rows(Layered* m, LayeredRun& r, const int* tokens, const Rows& rows, int pos0);
// final norm and output product of the given rows of the last layered_rows call (index null: all), {n, n_vocab}
void layered_rows_logits(Layered* m, LayeredRun& r, const int* index, int n, float* logits);

}  // namespace emelb
