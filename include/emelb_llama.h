/*
 * emelb_llama.h — device-resident Llama-architecture decode loop over the
 * kernels of emelb.h.
 *
 * Restates the caller side of the hot path: the reference's generator issues,
 * per token, the embedding row copy, per layer rms_norm -> Q/K/V mat-vecs ->
 * RoPE -> f16 KV store -> flash attention -> output projection + residual ->
 * rms_norm -> gate/up mat-vecs -> SwiGLU -> down projection + residual, then
 * the output norm and the logits mat-vec
 * (src/emel/text/generator/detail.hpp:3746-3840 compute_layer_attention_residual,
 *  :3852-3926 compute_layer_feed_forward, :3997-4033 compute_logits,
 *  :4860-4914 run_decode).  Here the whole token step is enqueued on the
 * context's stream (captured once as a CUDA graph) with every intermediate
 * kept in HBM; only the token id goes in and the next token id (or the logits)
 * comes out.
 */
#ifndef EMELB_LLAMA_H
#define EMELB_LLAMA_H

#include "emelb.h"
#include "emelb_window.h"

#ifdef __cplusplus
extern "C" {
#endif

typedef struct emelb_llama_config {
  int32_t n_layer;
  int32_t n_embd;
  int32_t n_head;
  int32_t n_head_kv;
  int32_t head_dim;
  int32_t n_ff;
  int32_t n_vocab;
  int32_t n_ctx;
  int32_t rope_dim;        /* rotated dims per head (n_rot) */
  int32_t rope_neox;       /* 0: adjacent pairs (Llama), 1: half-split pairs
                              (src/emel/text/generator/detail.hpp:38-50) */
  float rope_freq_base;
  float rms_eps;
  int32_t kv_block;        /* KV capacity is n_ctx rounded up to this (16 in the
                              reference, src/emel/memory/view.hpp:18,47-56) */
  int32_t shard_rank;      /* row sharding across GPUs: this rank ... */
  int32_t shard_count;     /* ... of this many (1 = unsharded).  With G > 1 the
                              context must have joined a G-rank exchange group
                              (emelb_comm_init) as this rank; n_head_kv, n_embd,
                              n_ff and n_vocab must be multiples of G; each
                              matrix is bound as this rank's contiguous row
                              interval (M/G rows: whole query/KV heads for
                              Q/K/V), the embedding table and norms whole.
                              Every rank calls decode/prefill/generate with
                              the same arguments; results are identical on
                              all ranks and equal to the unsharded session's
                              (src/emel/kernel/matmul/detail.hpp:36-57). */
} emelb_llama_config;

/* tensor roles for emelb_llama_bind; layer = -1 for the three model-level ones */
enum {
  EMELB_T_TOKEN_EMBD = 0,
  EMELB_T_OUTPUT_NORM = 1,
  EMELB_T_OUTPUT = 2,
  EMELB_T_ATTN_NORM = 3,
  EMELB_T_ATTN_Q = 4,
  EMELB_T_ATTN_K = 5,
  EMELB_T_ATTN_V = 6,
  EMELB_T_ATTN_OUT = 7,
  EMELB_T_FFN_NORM = 8,
  EMELB_T_FFN_GATE = 9,
  EMELB_T_FFN_UP = 10,
  EMELB_T_FFN_DOWN = 11
};

/* roles of layered sessions (emelb_llama_create_layers), beside EMELB_T_TOKEN_EMBD, EMELB_T_OUTPUT_NORM,
 * EMELB_T_OUTPUT, EMELB_T_ATTN_NORM (norm of the mixer's output), EMELB_T_ATTN_OUT, EMELB_T_FFN_NORM (norm of the
 * feed-forward's output) and EMELB_T_FFN_DOWN */
enum {
  EMELB_T_MIX_IN = 12,       /* the mixer's input projections stacked by rows: q|k|v (attention), q (a layer that
                                borrows keys and values), q|k|v|gate (linear) */
  EMELB_T_MIX_CONV = 13,     /* f32 [rows of MIX_IN][taps] */
  EMELB_T_MIX_NORM_Q = 14,   /* f32, over the whole query projection */
  EMELB_T_MIX_NORM_K = 15,   /* f32, over the whole key projection */
  EMELB_T_MIX_HEADS = 16,    /* f32 [n_head][n_head]: mixes the heads' attention weights */
  EMELB_T_MIX_NORM_OUT = 17, /* f32, over the concatenated heads of a linear mixer */
  EMELB_T_FFN_IN = 18,       /* gate|up stacked by rows */
  EMELB_T_FFN_IN_BIAS = 19,  /* f32, gate|up */
  EMELB_T_FFN_DOWN_BIAS = 20, /* f32 */
  EMELB_T_MIX_LATENT_NORM = 21, /* f32, kv_rank */
  EMELB_T_MIX_LATENT_UP = 22,   /* {kv_rank, n_head * (key_dim + value_dim)}: the latent's key rows of every head, then its value rows */
  EMELB_T_MIX_DECAY_LOG = 23,   /* f32, n_head: log of the delta rule's decay rate */
  EMELB_T_MIX_STEP_BIAS = 24,   /* f32, n_head: bias inside the decay's softplus */
  EMELB_T_LAYER_OUT = 25,       /* parallel layers: output projection and feed-forward's down projection side by side,
                                   {n_head * value_dim rounded up to 8 (zeros there) + n_ff, n_embd} */
  EMELB_T_LOOP_STEP = 26        /* model level, f32 {n_embd, loop_times}: added to the stream ahead of each pass */
};

typedef struct emelb_llama emelb_llama;

/* ---- layered sessions: decoders described layer by layer.  Each layer is a sequence mixer and, optionally, a
 * gated feed-forward.  How they meet the residual stream is the stack's arrangement (emelb_stack_config): by default
 * both read the stream itself and the norm (layer norm, weight only) is applied to what they return: x += norm1(mixer(x)),
 * x += norm2(ff(x)).  Weights are bf16, vectors f32; the residual stream, norms,
 * attention scores and weights, and recurrent state are f32.  A session of this kind works through the same entry
 * points as the block-quantized ones (prefill, decode, generate, the batch calls, sequences), with one difference:
 * its mixers carry state, so a call must continue a sequence at the position where the last one ended, or start it
 * again at position 0 (which forgets the sequence's state); any other position is EMELB_INVALID_REQUEST. */
enum {
  EMELB_MIXER_ATTENTION = 0, /* softmax attention: short causal convolution after the projections, query / key norm over
                                the whole projection, adjacent-pair RoPE on the first rope_dim dimensions, value norm
                                per head, sliding window that keeps the sequence's first tokens, mixing of the
                                heads' weights after the softmax; keys and values may be another layer's */
  EMELB_MIXER_LINEAR = 1,    /* linear attention with a fixed decay per head: S = decay S + k v^T, o = S^T q, with silu
                                on q, k and v; heads RMS-normed together and gated by sigmoid(gate) */
  EMELB_MIXER_LATENT = 2,    /* softmax attention whose keys and values are projections of one cached latent per token
                                (kv_rank values, RMS norm) and, with rope_dim > 0, one rotated key part shared by all heads:
                                head = key_dim unrotated + rope_dim rotated dimensions; sliding window; optional sigmoid gate
                                on the concatenated heads.  MIX_IN rows: q | gate (out_gate) | latent | rotated key part */
  EMELB_MIXER_DELTA = 3      /* gated delta rule: short causal convolution and silu on q, k, v; q and k unit vectors per head;
                                S = g S, u = beta (v - S^T k), S += k u^T, o = S^T q / sqrt(key_dim) with one decay g and one
                                step size beta per head and token; heads RMS-normed each and gated by silu(gate).  n_head_kv
                                query / key heads, n_head value heads.  MIX_IN rows: q | k | v | gate | beta | decay */
};
enum { EMELB_FF_SILU = 0, EMELB_FF_GELU_TANH = 1 };
typedef struct emelb_layer_config {
  int32_t mixer;
  int32_t n_head, n_head_kv; /* n_head_kv: attention only */
  int32_t key_dim, value_dim;
  int32_t conv_taps;         /* attention: taps of the short convolution on q, k and v; 0: none */
  int32_t norm_qk;           /* attention: 1 = query and key norm */
  int32_t norm_v;            /* attention: 1 = values divided by their root mean square per head */
  int32_t mix_heads;         /* attention: 1 = heads' weights mixed after the softmax */
  int32_t rope_dim;          /* rotated dimensions per head (even, 0: none) */
  float rope_freq_base;
  float attn_scale;
  int32_t window;            /* position i sees j with i - j < window (0: all) ... */
  int32_t keep_first;        /* ... and every j < keep_first */
  int32_t kv_from;           /* layer whose keys and values are used (-1: this layer's own) */
  int32_t n_ff;              /* 0: no feed-forward */
  const float* decay;        /* linear: n_head factors (read by the create call) */
  int32_t rope_half;         /* latent: 1 = dimension i turns with i + rope_dim / 2, 0 = with its neighbour */
  int32_t kv_rank;           /* latent: size of the latent */
  int32_t out_gate;          /* latent: 1 = heads multiplied by sigmoid(gate) */
  int32_t ff_act;            /* EMELB_FF_*: activation of the gate */
  int32_t ff_bias;           /* 1 = biases on gate | up and down */
} emelb_layer_config;

/* what the layers of a stack have in common */
enum {
  EMELB_STACK_POST_NORM = 0, /* x += norm1(mixer(x)); x += norm2(ff(x)) */
  EMELB_STACK_PARALLEL = 1   /* x += mixer(norm1(x)) + ff(norm2(x)), both of the same x */
};
enum { EMELB_NORM_LAYER = 0, EMELB_NORM_RMS = 1 };   /* of the stream; weight only */
typedef struct emelb_stack_config {
  int32_t arrangement;
  int32_t norm;
  int32_t loop_start, loop_stop, loop_times; /* layers loop_start .. loop_stop - 1 run loop_times times in a row with the same
                                weights, each pass with its own cache and state; loop_times 0: every layer runs once */
  int32_t loop_step;         /* 1 = EMELB_T_LOOP_STEP row t is added to the stream ahead of pass t */
  float logit_scale;         /* logits = logit_scale * output product ... */
  float logit_softcap;       /* ... then softcap * tanh(logits / softcap); 0: none */
} emelb_stack_config;

/* pure check of a configuration (no device needed): EMELB_OK or
 * EMELB_INVALID_REQUEST.  Beyond the plain range checks, a sharded layout
 * (shard_count G > 1, at most 8) must give every rank whole KV heads and whole
 * rows, and every row interval that is joined across ranks — n_head*head_dim/G,
 * n_embd/G, n_ff/G and n_vocab/G f32 values — must be a multiple of 4 values
 * (joins move 16-byte units).  emelb_llama_create applies it first. */
EMELB_API uint32_t emelb_llama_check_config(const emelb_llama_config* cfg);

/* allocates activations, the f16 KV cache in the flash layout
 * [layer][kv_head][capacity][head_dim]
 * (src/emel/text/generator/detail.hpp:3010-3048) and the RoPE table */
EMELB_API uint32_t emelb_llama_create(emelb_ctx* ctx, const emelb_llama_config* cfg,
                                      emelb_llama** out);
EMELB_API uint32_t emelb_llama_destroy(emelb_llama* s);

/* a layered session.  Of cfg, n_layer, n_embd, n_vocab, n_ctx, rms_eps (every norm's eps) and kv_block are used and
 * shard_count must be 1.  float32 = 1: activations, products and caches in f32 throughout (no reduced-precision
 * matrix mode); 0: matrix operands and the key / value cache in bf16 with f32 accumulation.
 * Matrices are bound as {K, M} views of type EMELB_BF16 whose row stride is a multiple of 16 bytes, with zeros
 * between K and the stride; vectors as EMELB_F32 at a 16-byte boundary. */
EMELB_API uint32_t emelb_llama_check_layers(const emelb_llama_config* cfg, const emelb_layer_config* layers);
EMELB_API uint32_t emelb_llama_create_layers(emelb_ctx* ctx, const emelb_llama_config* cfg,
                                             const emelb_layer_config* layers, int32_t float32, emelb_llama** out);
/* the same with the stack described; emelb_llama_create_layers is post-norm with layer norm, no loop, plain logits */
EMELB_API uint32_t emelb_llama_check_stack(const emelb_llama_config* cfg, const emelb_stack_config* stack,
                                           const emelb_layer_config* layers);
EMELB_API uint32_t emelb_llama_create_stack(emelb_ctx* ctx, const emelb_llama_config* cfg, const emelb_stack_config* stack,
                                            const emelb_layer_config* layers, int32_t float32, emelb_llama** out);

/* binds one tensor (replaces bind_tensor_rows / make_src_view,
 * src/emel/text/generator/detail.hpp:788-817, 1886-1919): a {K, M} view of
 * native blocks (matrices) or f32 (norm vectors) whose data is a device
 * pointer or a host pointer inside a resident span */
EMELB_API uint32_t emelb_llama_bind(emelb_llama* s, int32_t layer, int32_t role,
                                    const emelb_view* tensor);

/* one decode step at `position` (replaces run_decode).  logits_out (n_vocab
 * f32, host or device) and token_out (greedy argmax, lowest id on ties) may
 * each be null; with logits_out null the logits are never materialised
 * (op_mul_mat_argmax route, src/emel/text/generator/detail.hpp:4035-4060). */
EMELB_API uint32_t emelb_llama_decode(emelb_llama* s, int32_t token, int32_t position,
                                      float* logits_out, int32_t* token_out);

/* feeds `n` prompt tokens at positions start_pos.. without computing logits:
 * fills their KV rows.  The reference's x86 prefill walks the prompt one token
 * at a time (src/emel/text/generator/detail.hpp:4064-4092).  With the fast
 * attention (mode 0) the prompt is processed in batches of up to 2048 tokens
 * (emelb_llama_set_prefill_batch) instead: per token the same arithmetic except the attention, which is an f32
 * online softmax over the batch (emelb_flash_attn_batch).  Sharded sessions do
 * the same when their context has a communicator (emelb_comm_init), joining the
 * ranks' row intervals of every product by all-gather.  The reference-order
 * attention modes walk token by token. */
EMELB_API uint32_t emelb_llama_prefill(emelb_llama* s, const int32_t* tokens, int32_t n,
                                       int32_t start_pos);

/* emelb_llama_prefill that also returns logits: want[0..n_want) are places among the n tokens (ascending), and
 * logits_out (host) gets n_want rows of n_vocab f32.  Unsharded sessions. */
EMELB_API uint32_t emelb_llama_prefill_logits(emelb_llama* s, const int32_t* tokens, int32_t n, int32_t start_pos,
                                              const int32_t* want, int32_t n_want, float* logits_out);

/* layered sessions: the residual stream after every layer run (a looped layer counts once per pass) for the tokens of the
 * last prefill batch is copied to `out` (device or host, {layer runs, tokens, n_embd} f32, tokens <= max_tokens) by the following prefill calls; null
 * turns it off (diagnostics). */
EMELB_API uint32_t emelb_llama_trace_layers(emelb_llama* s, float* out, int32_t max_tokens);

/* prompt tokens per batch of emelb_llama_prefill: default 2048; 0 or 1 walks the
 * prompt token by token (what the reference does); the first batched prompt sizes
 * the session's batch buffers, later values are clamped to them */
EMELB_API uint32_t emelb_llama_set_prefill_batch(emelb_llama* s, int32_t max_tokens);

/* greedy generation of `n` tokens with the token fed back on the device: no
 * host round trip between steps; tokens_out (host) is written at the end */
EMELB_API uint32_t emelb_llama_generate(emelb_llama* s, int32_t first_token,
                                        int32_t start_pos, int32_t n, int32_t* tokens_out);

/* Row-sharded sessions on one node: the joins of the ranks' row intervals can run as
 * peer stores over NVLink instead of NCCL all-gathers (one small kernel per join).
 * Each rank exports a handle of its exchange arena (the joined vectors live in it),
 * the caller all-gathers the G handles, and each rank attaches them (rank order,
 * G x EMELB_EXCHANGE_HANDLE_BYTES).  Attach on every rank and synchronise the ranks
 * before the first step (a join waits at most 10 s for a peer, then the step fails with
 * EMELB_INTERNAL_ERROR at the next emelb_sync);
 * without it the session keeps using the context's NCCL communicator.  No reference
 * counterpart beyond the lane join of src/emel/kernel/matmul/actions.hpp:108-136. */
#define EMELB_EXCHANGE_HANDLE_BYTES 64
EMELB_API uint32_t emelb_llama_exchange_export(emelb_llama* s, uint8_t* handle_out,
                                               uint64_t handle_bytes);
EMELB_API uint32_t emelb_llama_exchange_attach(emelb_llama* s, const uint8_t* handles,
                                               uint64_t handles_bytes);
/* unmaps the peers' arenas (the session falls back to NCCL joins).  Tear-down order
 * across ranks: every rank detaches, the caller synchronises the ranks, then the
 * sessions are destroyed — no arena is freed while a peer still maps it. */
EMELB_API uint32_t emelb_llama_exchange_detach(emelb_llama* s);

/* ---- several sequences decoded together (batch decode).  A session holds n_seq KV caches (default 1;
 * emelb_llama_set_sequences reallocates and clears them).  The one-sequence entry points above (prefill, decode,
 * generate) work on the sequence chosen by emelb_llama_select_sequence (default 0), so a caller fills each
 * sequence's cache with its prompt and then steps all of them together:
 *   decode_batch   one step: sequence j (0 <= j < n_seq) takes tokens[j] at positions[j]; logits_out (optional,
 *                  host, {n_vocab, n_seq} with the sequence index fastest -- op_mul_mat's result layout) and
 *                  tokens_out (optional, host, the greedy next id per sequence);
 *   generate_batch n_steps greedy steps fed back on the device, one CUDA-graph replay per step;
 *                  tokens_out[step * n_seq + j].
 * Column j of every product is computed with the arithmetic of the one-sequence step (same block order, same
 * rotation, split-KV attention with the same split count), so each sequence gets exactly the tokens and logits
 * it gets when decoded alone.  Needs attention mode 0; EMELB_UNSUPPORTED_OP otherwise.  The reference's generator
 * decodes one sequence per session (src/emel/text/generator/detail.hpp:4860-4914); this is that loop over
 * several sessions' worth of state with the weights streamed once per step. */
EMELB_API uint32_t emelb_llama_set_sequences(emelb_llama* s, int32_t n_seq);
EMELB_API uint32_t emelb_llama_select_sequence(emelb_llama* s, int32_t seq);
EMELB_API uint32_t emelb_llama_decode_batch(emelb_llama* s, const int32_t* tokens, const int32_t* positions, int32_t n_seq,
                                            float* logits_out, int32_t* tokens_out);
EMELB_API uint32_t emelb_llama_generate_batch(emelb_llama* s, const int32_t* first_tokens, const int32_t* start_positions,
                                              int32_t n_seq, int32_t n_steps, int32_t* tokens_out);
EMELB_API uint32_t emelb_llama_batch_launches_per_step(const emelb_llama* s, int32_t* out);

/* Row-sharded sessions with every peer attached: where a layer's products all take the streaming kernel, its four
 * joins run inside the kernels either side of them -- the producing kernel (attention merge, output projection,
 * SwiGLU, down projection) stores its rows into every rank's copy of the vector and raises a flag, the consuming
 * product waits for the flags and quantizes the joined f32 vector in its prologue -- instead of one join kernel
 * each.  on = 0 (default): one join kernel per join; on = 1: inside the neighbouring kernels (232 instead of 423
 * launches per token at the 8B shape; measured no faster on 2 GPUs and slower on 4, hence not the default).  Same
 * result bit for bit either way. */
EMELB_API uint32_t emelb_llama_set_join_fusion(emelb_llama* s, int32_t on);

/* Layers streamed from host memory (models whose layers do not fit the HBM left for weights).  `w` is a bound,
 * streaming emelb_window on the session's context with one layer descriptor per model layer.  After this call
 * emelb_llama_bind accepts, for a layer tensor, a view whose `data` is not resident but is the address of one of that
 * layer's extents inside the window's source (same byte size): the tensor is then read from the slot the window
 * hands out for the layer.  Resident and streamed tensors may be mixed.  Each layer pass of a step, of a prompt batch
 * and of a batch step acquires its layer once, so the next layers cross PCIe while the current one computes; steps
 * run as plain launches instead of replayed graphs.  Same results bit for bit as the resident session.  Unsharded
 * sessions only.  The window must stay bound while tensors of the session are bound through it; w = null detaches
 * (refused while streamed tensors are bound). */
EMELB_API uint32_t emelb_llama_set_window(emelb_llama* s, emelb_window* w);

/* How a decode step is enqueued.  0 (default): the chain of per-operation
 * launches.  1: where the session qualifies (unsharded, Q4_K layer matrices with
 * K a multiple of 2048, head size 128, adjacent-pair RoPE, fast attention mode),
 * all layers of a token run as ONE persistent kernel, one CTA per SM, with grid
 * barriers between the phases of a layer and producer warps that keep the
 * weights streaming across them; sessions that do not qualify keep the chain.
 * Both give the same numbers bit for bit.  No reference counterpart (its
 * generator calls the kernel actor once per operation,
 * src/emel/text/generator/detail.hpp:3746-3926). */
EMELB_API uint32_t emelb_llama_set_step_mode(emelb_llama* s, int32_t mode);

/* Phase profile of the one-kernel step (diagnostics, like the reference's
 * capture_diagnostics counters): runs the layers of one decode step at
 * (token, position) — the KV row of `position` is written as in a normal step,
 * no logits are produced — and returns, for each layer, 16 nanosecond stamps
 * taken by one CTA: 0 layer start, 1 Q/K/V input staged, 2 Q/K/V products done,
 * 3/5/8/11/14 after the grid barriers, 4 attention done, 6 output-projection
 * input staged, 7 output projection done, 9 gate/up input staged, 10 gate/up
 * done, 12 SwiGLU staged, 13 down projection done.  stamps_count >= 16 * n_layer.
 * EMELB_UNSUPPORTED_OP when the session does not qualify for the one-kernel step. */
EMELB_API uint32_t emelb_llama_decode_profile(emelb_llama* s, int32_t token, int32_t position,
                                              uint64_t* stamps_ns, uint64_t stamps_count);

/* kernels launched per decode step (for launch accounting) */
EMELB_API uint32_t emelb_llama_launches_per_token(const emelb_llama* s, int32_t* out);

#ifdef __cplusplus
}
#endif
#endif /* EMELB_LLAMA_H */
