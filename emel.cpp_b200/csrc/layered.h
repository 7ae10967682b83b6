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

enum Act : int { ACT_NONE = 0, ACT_SILU_SIGMOID = 1, ACT_GLU = 2, ACT_GLU_GELU = 3, ACT_SOFTCAP = 4 };
inline bool is_glu(int act) { return act == ACT_GLU || act == ACT_GLU_GELU; }

// ---- linear.cu: products with bf16 weights
// y {rows, M} = act(x W^T + bias).  ACT_SILU_SIGMOID: silu on features below act_split, sigmoid on the others.
// ACT_GLU: W holds M gate rows, then M up rows (bias likewise); y = silu(gate) * up.  ACT_GLU_GELU: gelu (tanh form).
// ACT_SOFTCAP: y = softcap tanh(out_scale y / softcap), out_scale y where softcap is 0.
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
  float out_scale = 1.0f, softcap = 0.0f;
  // many rows, bf16 outputs: features from `tail` on are stored as f32 instead, feature f of row r at
  // tail_y[r * tail_ld + f - tail]
  int tail = 0x7fffffff;
  float* tail_y = nullptr;
  int64_t tail_ld = 0;
};
// what the one-row kernel does to its input before the product, in every block
enum Prologue : int {
  PRO_PLAIN = 0,       // x
  PRO_EMBED = 1,       // row *token of the bf16 table, also written to x_out
  PRO_RESIDUAL = 2,    // x + layer_norm(y) * norm_w, also written to x_out
  PRO_RESIDUAL_NORM = 3,  // layer_norm(that) * norm2_w
  PRO_RMS_GATE = 4,    // rms_norm(x) * norm_w * gate
  PRO_PRENORM = 5,     // norm(x + y) * norm_w, and * norm2_w for the second matrix; x + y also written to x_out
};
struct VecArgs {
  int pro;
  int rms;                 // the norm of PRO_RESIDUAL* and PRO_PRENORM: 0 layer norm, 1 RMS norm
  const float* x;
  const float* y;          // PRO_RESIDUAL*, PRO_PRENORM (null: none)
  const float* step;       // PRO_EMBED, PRO_RESIDUAL, PRO_PRENORM (null: none): added to the stream
  const float* norm_w;
  const float* norm2_w;
  const float* gate;
  float eps;
  float* x_out;
  const __nv_bfloat16* table;   // PRO_EMBED; PRO_PRENORM: stands for x where it is set
  int64_t table_ld;
  const int* token;
  float* out;
  Bf16Matrix w2;           // PRO_PRENORM: a second matrix of the same K (w null: none), act2 into out2
  const float* bias2;
  int act2;
  float* out2;
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
// rms: 0 layer norm, 1 RMS norm; step (optional): added to the stream after that
template <class T>
cudaError_t launch_embed_rows_bf16(const __nv_bfloat16* table, int64_t ld, const int* tokens, const float* step, int rows, int width, float* x,
                                   T* xb, int64_t ldb, cudaStream_t st);
// x += norm(y) * w; keep (optional) = a copy of x; x += step; xb = T(x)
template <class T>
cudaError_t launch_residual_norm(float* x, const float* y, const float* w, int rms, float eps, int rows, int width, T* xb, int64_t ldb, float* keep,
                                 const float* step, cudaStream_t st);
// out row r = T(norm(x row index[r]) * w)   (index null: r)
template <class T>
cudaError_t launch_norm_rows(const float* x, const int* index, const float* w, int rms, float eps, int rows, int width, T* out, int64_t ldo,
                             cudaStream_t st);
// the stream in front of a parallel layer: x = table row of the token, or x += y; keep (optional) = a copy; x += step;
// h1 = T(norm(x) * w1), h2 = T(norm(x) * w2) (each optional)
struct PrenormArgs {
  float* x;
  const float* y;
  const __nv_bfloat16* table;   // null: x is there already
  int64_t table_ld;
  const int* tokens;
  float* keep;
  const float* step;
  const float *w1, *w2;
  int rms;
  float eps;
  int rows, width;
  void *h1, *h2;
  int64_t ldh;
};
template <class T>
cudaError_t launch_prenorm_rows(const PrenormArgs& a, cudaStream_t st);
template <class T>
cudaError_t launch_rms_gate(const float* o, const float* w, const T* gate, int64_t ldg, float eps, int rows, int width, T* out, int64_t ldo,
                            cudaStream_t st);
// gate|up {rows, 2 ff} -> act(gate) * up (ACT_GLU, ACT_GLU_GELU)
cudaError_t launch_glu_rows(const float* gu, int rows, int ff, int act, float* out, int64_t ldo, cudaStream_t st);

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

// ---- latent_attention.cu: softmax attention over one cached latent per token
constexpr int kLatentRows = 64;   // rows per launch of the row-by-row route (scratch)
struct LatentArgs {
  void* proj;              // T rows: q {heads, dim + rot} | gate {heads, vdim}
  int64_t ldp;
  const float* down;       // rows: latent before its norm (rank) | key part before its rotation (rot)
  int64_t ldd;
  int heads, dim, rot, vdim, rank;
  int gate_at;             // feature the gate starts at (0: no gate)
  const float* norm;       // [rank]
  float eps;
  const float *rope_cos, *rope_sin;   // [position][rot / 2]
  int rope_half;           // pairs: 1 (i, i + rot / 2), 0 (2 i, 2 i + 1)
  Bf16Matrix up;           // key rows of every head, then value rows
  void* cache;             // T [sequence][capacity][width]: latent, zeros to rank_pad, rotated key part, zeros
  int64_t capacity;
  int rank_pad, width;
  float scale;
  int window, max_visible;
  float* qlat;             // scratch {kLatentRows, heads, width}
  float* stats;            // scratch
  uint64_t stats_floats;
  float* part;             // scratch
  uint64_t part_floats;
  __nv_bfloat16* kv;       // prompts: keys and values of the visible positions {keys, heads * (dim + vdim)}
  int64_t kv_rows, kv_ld;
};
// latents and key parts of the rows into the cache, scores against the latents themselves (the key rows of `up` meet
// the query first), values from the weighted latents.  TC = cache type, TP = type of proj, TO = type of out
template <class TC, class TP, class TO>
cudaError_t launch_latent_rows(const LatentArgs& a, const Rows& rows, TO* out, int64_t ldo, int sm_count, bool pdl, cudaStream_t st, int* launches);
// prompts on the tensor cores: keys and values of every visible position are projected first (upmap: `up`)
bool latent_prompt_supported(const LatentArgs& a, int rows);
cudaError_t launch_latent_prompt(const LatentArgs& a, const TmaMap& upmap, const Rows& rows, int pos0, __nv_bfloat16* out, int64_t ldo, int* status,
                                 cudaStream_t st, int* launches);

// ---- delta.cu: gated delta rule
struct DeltaArgs {
  const void* proj;        // T rows: q | k {kv_heads, dim} | v | gate {heads, vdim}
  int64_t ldp;
  const float* gates;      // rows: step size (heads) | decay (heads), before their activations
  int64_t ldg;
  const float* conv;       // [taps][channels], channels = q | k | v
  int taps;
  float* conv_state;       // ring [sequence][taps][channels]: the projections of position p at entry p % taps
  const float *decay_log, *step_bias;   // [heads]
  const float* norm;       // [vdim]
  float eps;
  int heads, kv_heads, dim, vdim;
  float* state;            // [sequence][heads][dim][vdim]
  // prompts: scratch
  void* qkv;               // T rows after convolution and silu, ldc elements apart
  int64_t ldc;
  float* scalars;          // rows: 1 / |q| / sqrt(dim), 1 / |k| (kv_heads each) | beta | log decay (heads each)
  float* chunks;           // per (chunk, head) what the tensor-core route needs (delta_chunk_floats each)
  float* o;                // {rows, heads * vdim}
  __host__ __device__ int channels() const { return 2 * kv_heads * dim + heads * vdim; }
  __host__ __device__ int scalar_count() const { return 2 * kv_heads + 2 * heads; }
};
// one token of each sequence, everything from the projections to the gated heads
template <class TP, class TO>
cudaError_t launch_delta_step(const DeltaArgs& a, const Rows& rows, TO* out, int64_t ldo, bool pdl, cudaStream_t st);
// a prompt: convolution and scalars, the recurrence (token by token, or chunks on the tensor cores), norm and gate
template <class T>
cudaError_t launch_delta_prompt(const DeltaArgs& a, const Rows& rows, T* out, int64_t ldo, int sm_count, cudaStream_t st, int* launches);
bool delta_chunks_supported(const DeltaArgs& a);
size_t delta_chunk_floats();                 // scratch per (chunk, head)
int delta_chunks(int rows);

// ---- layered.cu: the model object
struct Layered;
struct LayeredRun {
  cudaStream_t st;
  int launches = 0;
  bool ok = true;
};
emelb_stack_config layered_default_stack();
uint32_t layered_check(const emelb_llama_config& cfg, const emelb_stack_config& stack, const emelb_layer_config* layers);
Layered* layered_create(emelb_ctx* c, const emelb_llama_config& cfg, const emelb_stack_config& stack, const emelb_layer_config* layers, bool f32);
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
