// The model object of a layered session (layered.h): per layer weights, caches and recurrent state of every sequence,
// activation buffers, and the two ways through the layers -- one token (fused one-row products) and many rows.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <map>
#include <new>
#include <utility>
#include <vector>

#include "ctx.h"
#include "layered.h"

namespace emelb {
const void* ctx_resolve_weights(emelb_ctx* c, const void* p);  // api.cu
bool ctx_cuda_ok(emelb_ctx* c, cudaError_t e);

namespace {

using bf16 = __nv_bfloat16;
int64_t pad8(int64_t n) { return (n + 7) / 8 * 8; }

struct LayerW {
  Bf16Matrix in, o, ff_in, ff_down, up, out;   // out: o and ff_down side by side (parallel layers)
  TmaMap in_map, o_map, ff_in_map, ff_down_map, up_map, out_map;
  const float *conv = nullptr, *norm_q = nullptr, *norm_k = nullptr, *talk = nullptr, *norm_out = nullptr, *norm_latent = nullptr;
  const float *decay_log = nullptr, *step_bias = nullptr;
  const float *norm1 = nullptr, *norm2 = nullptr, *ff_in_bias = nullptr, *ff_down_bias = nullptr;
};

struct LayerS {
  emelb_layer_config cfg{};
  int in_rows = 0;              // rows of the stacked input projections
  float* decay = nullptr;       // linear
  const float *rope_cos = nullptr, *rope_sin = nullptr;
  LayerW w;
  XMaps o_x{}, h_x{}, out_x{};  // the operand buffers as this layer's products read them
  bool own_kv() const { return cfg.kv_from < 0; }
  bool attention() const { return cfg.mixer == EMELB_MIXER_ATTENTION; }
  bool linear() const { return cfg.mixer == EMELB_MIXER_LINEAR; }
  bool latent() const { return cfg.mixer == EMELB_MIXER_LATENT; }
  bool delta() const { return cfg.mixer == EMELB_MIXER_DELTA; }
  int out_dim() const { return cfg.n_head * cfg.value_dim; }
  // columns of the side-by-side output matrix
  int joint_dim() const { return (int)pad8(out_dim()) + cfg.n_ff; }
  int linear_gate_at() const { return 2 * cfg.n_head * cfg.key_dim + cfg.n_head * cfg.value_dim; }
  int q_dim() const { return cfg.n_head * (cfg.key_dim + (latent() ? cfg.rope_dim : 0)); }
  int conv_channels() const { return delta() ? 2 * cfg.n_head_kv * cfg.key_dim + out_dim() : in_rows; }
  // first of the projected features that stay f32 in bf16 batches
  int tail_at() const { return latent() ? in_rows - cfg.kv_rank - cfg.rope_dim : delta() ? in_rows - 2 * cfg.n_head : in_rows; }
  int rank_pad() const { return (int)pad8(cfg.kv_rank); }
  int cache_width() const { return rank_pad() + (int)pad8(cfg.rope_dim); }
  int up_rows() const { return cfg.n_head * (cfg.key_dim + cfg.value_dim); }
};

// a layer's turn in the stack, with the cache and state of its pass
struct RunS {
  int layer = 0;
  int pass = -1;                // the pass that starts with this run, -1: none does
  int kv_run = -1;              // attention on another layer's keys and values: the run that owns them
  void *k = nullptr, *v = nullptr;   // latent: the latents in k
  float* conv_state = nullptr;
  float* state = nullptr;
};

int in_rows_of(const emelb_layer_config& l) {
  switch (l.mixer) {
    case EMELB_MIXER_LINEAR: return 2 * l.n_head * l.key_dim + 2 * l.n_head * l.value_dim;
    case EMELB_MIXER_LATENT: return l.n_head * (l.key_dim + l.rope_dim + (l.out_gate ? l.value_dim : 0)) + l.kv_rank + l.rope_dim;
    case EMELB_MIXER_DELTA: return 2 * l.n_head_kv * l.key_dim + 2 * l.n_head * l.value_dim + 2 * l.n_head;
    default: return l.n_head * l.key_dim + (l.kv_from < 0 ? l.n_head_kv * (l.key_dim + l.value_dim) : 0);
  }
}

}  // namespace

struct Layered {
  emelb_ctx* c = nullptr;
  emelb_llama_config cfg{};
  emelb_stack_config stack{};
  bool f32 = false;
  std::vector<LayerS> layers;
  std::vector<RunS> runs;
  Bf16Matrix embed, head;
  TmaMap head_map;
  const float *final_norm = nullptr, *loop_step = nullptr;
  int64_t capacity = 0;
  int n_seq = 0;
  std::vector<void*> owned, seq_owned, row_owned;
  // one token
  float *vx[2] = {nullptr, nullptr}, *vproj = nullptr, *vmix = nullptr, *vh = nullptr, *vy = nullptr;
  void* vq = nullptr;
  float* qlat = nullptr;        // latent queries of kLatentRows rows
  // rows
  int row_cap = 0;
  float *x = nullptr, *y = nullptr, *proj = nullptr, *lin = nullptr, *gu = nullptr;
  void *xb = nullptr, *xb2 = nullptr, *projb = nullptr, *q = nullptr, *mix = nullptr, *h = nullptr, *nb = nullptr;
  XMaps xb_x{}, xb2_x{}, nb_x{};
  float* tail = nullptr;        // the projections' f32 features
  bf16* kv = nullptr;           // latent prompts: keys and values of the visible positions
  size_t kv_elems = 0;
  void* qkv = nullptr;          // delta prompts: convolved q | k | v, the tokens' scalars, per-chunk operands
  float *delta_scalars = nullptr, *delta_chunk = nullptr;
  // attention scratch
  float* lin_local = nullptr;
  float *scores = nullptr, *stats = nullptr, *part = nullptr;
  uint64_t scores_floats = 0, stats_floats = 0, part_floats = 0;
  float* trace_out = nullptr;
  float* trace_dev = nullptr;
  int trace_tokens = 0;

  size_t operand_bytes() const { return f32 ? 4 : 2; }
  bool parallel() const { return stack.arrangement == EMELB_STACK_PARALLEL; }
  int rms() const { return stack.norm == EMELB_NORM_RMS; }
  // what is added to the stream ahead of run i (null: nothing)
  const float* step_before(size_t i) const {
    return loop_step && i < runs.size() && runs[i].pass >= 0 ? loop_step + (int64_t)runs[i].pass * cfg.n_embd : nullptr;
  }
};

namespace {

bool alloc(std::vector<void*>& list, void** p, size_t bytes) {
  if (cudaMalloc(p, (bytes + 255) & ~size_t(255)) != cudaSuccess) {
    cudaGetLastError();
    *p = nullptr;
    return false;
  }
  list.push_back(*p);
  return true;
}
template <class T>
bool alloc_n(std::vector<void*>& list, T** p, size_t count) {
  return alloc(list, reinterpret_cast<void**>(p), sizeof(T) * count);
}
void free_all(std::vector<void*>& list) {
  for (void* p : list) cudaFree(p);
  list.clear();
}

int max_visible(const Layered* m, const emelb_layer_config& l) {
  const int64_t v = l.window > 0 ? (int64_t)l.window + l.keep_first : m->cfg.n_ctx;
  return (int)std::min<int64_t>(v, m->cfg.n_ctx);
}

AttnInArgs attn_in_args(const Layered* m, const LayerS& l, const RunS& run, const float* proj, void* q) {
  const emelb_layer_config& g = l.cfg;
  AttnInArgs a{};
  a.proj = proj;
  a.channels = l.in_rows;
  a.conv = l.w.conv;
  a.taps = g.conv_taps > 0 ? g.conv_taps : 1;
  a.conv_state = run.conv_state;
  a.norm_q = l.w.norm_q;
  a.norm_k = l.w.norm_k;
  a.norm_v = g.norm_v;
  a.eps = m->cfg.rms_eps;
  a.heads = g.n_head;
  a.kv_heads = g.n_head_kv;
  a.dim = g.key_dim;
  a.vdim = g.value_dim;
  a.dim_pad = (int)pad8(g.key_dim);
  a.vdim_pad = (int)pad8(g.value_dim);
  a.own_kv = l.own_kv();
  a.rope_cos = l.rope_cos;
  a.rope_sin = l.rope_sin;
  a.rope_dim = g.rope_dim;
  a.q = q;
  a.k = run.k;
  a.v = run.v;
  a.capacity = m->capacity;
  return a;
}

MixAttnArgs mix_args(const Layered* m, const LayerS& l, const RunS& run, const void* q) {
  const emelb_layer_config& g = l.cfg;
  const RunS& kv = l.own_kv() ? run : m->runs[run.kv_run];
  MixAttnArgs a{};
  a.q = q;
  a.k = kv.k;
  a.v = kv.v;
  a.capacity = m->capacity;
  a.heads = g.n_head;
  a.kv_heads = g.n_head_kv;
  a.dim_pad = (int)pad8(g.key_dim);
  a.vdim = g.value_dim;
  a.vdim_pad = (int)pad8(g.value_dim);
  a.scale = g.attn_scale;
  a.window = g.window;
  a.keep_first = g.keep_first;
  a.talk = l.w.talk;
  a.scores = m->scores;
  a.scores_floats = m->scores_floats;
  a.stats = m->stats;
  a.stats_floats = m->stats_floats;
  a.part = m->part;
  a.part_floats = m->part_floats;
  a.max_visible = max_visible(m, g);
  return a;
}

LinAttnArgs lin_args(const Layered* m, const LayerS& l, const RunS& run, int64_t ldx, float* out) {
  const emelb_layer_config& g = l.cfg;
  return LinAttnArgs{ldx, g.n_head, g.key_dim, g.value_dim, l.decay, run.state, out, m->lin_local};
}

LatentArgs latent_args(const Layered* m, const LayerS& l, const RunS& run, void* proj, int64_t ldp, const float* down, int64_t ldd) {
  const emelb_layer_config& g = l.cfg;
  LatentArgs a{};
  a.proj = proj;
  a.ldp = ldp;
  a.down = down;
  a.ldd = ldd;
  a.heads = g.n_head;
  a.dim = g.key_dim;
  a.rot = g.rope_dim;
  a.vdim = g.value_dim;
  a.rank = g.kv_rank;
  a.gate_at = g.out_gate ? l.q_dim() : 0;
  a.norm = l.w.norm_latent;
  a.eps = m->cfg.rms_eps;
  a.rope_cos = l.rope_cos;
  a.rope_sin = l.rope_sin;
  a.rope_half = g.rope_half;
  a.up = l.w.up;
  a.cache = run.k;
  a.capacity = m->capacity;
  a.rank_pad = l.rank_pad();
  a.width = l.cache_width();
  a.scale = g.attn_scale;
  a.window = g.window;
  a.max_visible = max_visible(m, g);
  a.qlat = m->qlat;
  a.stats = m->stats;
  a.stats_floats = m->stats_floats;
  a.part = m->part;
  a.part_floats = m->part_floats;
  a.kv = m->kv;
  a.kv_ld = pad8(l.up_rows());
  a.kv_rows = (int64_t)m->kv_elems / a.kv_ld;
  return a;
}

DeltaArgs delta_args(const Layered* m, const LayerS& l, const RunS& run, const void* proj, int64_t ldp, const float* gates, int64_t ldg) {
  const emelb_layer_config& g = l.cfg;
  DeltaArgs a{};
  a.proj = proj;
  a.ldp = ldp;
  a.gates = gates;
  a.ldg = ldg;
  a.conv = l.w.conv;
  a.taps = g.conv_taps;
  a.conv_state = run.conv_state;
  a.decay_log = l.w.decay_log;
  a.step_bias = l.w.step_bias;
  a.norm = l.w.norm_out;
  a.eps = m->cfg.rms_eps;
  a.heads = g.n_head;
  a.kv_heads = g.n_head_kv;
  a.dim = g.key_dim;
  a.vdim = g.value_dim;
  a.state = run.state;
  a.qkv = m->qkv;
  a.ldc = pad8(a.channels());
  a.scalars = m->delta_scalars;
  a.chunks = m->delta_chunk;
  a.o = m->lin;
  return a;
}

bool check(Layered* m, LayeredRun& r, cudaError_t e, int launches = 1) {
  r.launches += launches;
  r.ok = ctx_cuda_ok(m->c, e) && r.ok;
  return r.ok;
}

bool x_maps(XMaps* x, const void* base, int64_t rows, int64_t k, int64_t ld) {
  const bf16* b = static_cast<const bf16*>(base);
  return encode_bf16_map(&x->narrow, b, rows, k, ld, kGemmTokenBox) && encode_bf16_map(&x->wide, b, rows, k, ld, 128);
}

// y = act(x W^T + bias) over rows: bf16 operands on the tensor cores, or f32
void linear(Layered* m, LayeredRun& r, const LinearArgs& a, const TmaMap& wmap, const void* x, int64_t ldx, const XMaps& xm, float* y, bf16* yb,
            int64_t ldy) {
  if (m->f32) check(m, r, launch_linear_f32(a, static_cast<const float*>(x), ldx, y, ldy, r.st));
  else check(m, r, launch_gemm_bf16(a, wmap, xm, y, yb, ldy, m->c->status_word(), r.st));
}

// the mixer of one layer run over rows: in (operands, ld pad8(n_embd)) -> heads {rows, out_dim} at out
template <class T>
void mixer_rows(Layered* m, LayeredRun& r, const LayerS& l, const RunS& run, const Rows& rows, int pos0, const T* in, const XMaps& in_x, T* out, int64_t ldo) {
  const int n = rows.n, od = l.out_dim();
  const int64_t ldx = pad8(m->cfg.n_embd);
  if (l.attention()) {
    linear(m, r, LinearArgs{l.w.in, nullptr, ACT_NONE, 0, n}, l.w.in_map, in, ldx, in_x, m->proj, nullptr, l.in_rows);
    const AttnInArgs in_args = attn_in_args(m, l, run, m->proj, m->q);
    check(m, r, launch_attn_in<T>(in_args, rows, r.st));
    if (rows.prompt && in_args.conv && in_args.taps > 1) check(m, r, launch_conv_state(in_args, rows, r.st));
    const MixAttnArgs a = mix_args(m, l, run, m->q);
    if (!m->f32 && rows.prompt && mix_attention_prompt_supported(a))
      check(m, r, launch_mix_attention_prompt(a, rows, pos0, reinterpret_cast<bf16*>(out), ldo, r.st, &r.launches), 0);
    else
      check(m, r, (launch_mix_attention_rows<T, T>(a, rows, out, ldo, m->c->sm_count, r.st, &r.launches)), 0);
    return;
  }
  // operands of the following kernels; the last features of latent and delta projections stay f32
  const int64_t ldp = pad8(l.in_rows);
  T* proj = static_cast<T*>(m->projb);
  LinearArgs la{l.w.in, nullptr, l.linear() ? ACT_SILU_SIGMOID : ACT_NONE, l.linear() ? l.linear_gate_at() : 0, n};
  const float* tail = static_cast<const float*>(m->projb) + l.tail_at();
  int64_t tail_ld = ldp;
  if (!m->f32) {
    la.tail = l.tail_at();
    la.tail_y = m->tail;
    la.tail_ld = l.in_rows - l.tail_at();
    tail = m->tail;
    tail_ld = la.tail_ld;
  }
  linear(m, r, la, l.w.in_map, in, ldx, in_x, reinterpret_cast<float*>(m->projb), m->f32 ? nullptr : static_cast<bf16*>(m->projb), ldp);
  if (l.linear()) {
    const LinAttnArgs a = lin_args(m, l, run, ldp, m->lin);
    if (!m->f32 && rows.prompt && linear_attention_prompt_supported(a))
      check(m, r, launch_linear_attention_prompt(a, reinterpret_cast<const bf16*>(proj), rows, m->c->sm_count, r.st, &r.launches), 0);
    else
      check(m, r, launch_linear_attention_rows<T>(a, proj, rows, r.st));
    check(m, r, launch_rms_gate<T>(m->lin, l.w.norm_out, proj + l.linear_gate_at(), ldp, m->cfg.rms_eps, n, od, out, ldo, r.st));
  } else if (l.latent()) {
    const LatentArgs a = latent_args(m, l, run, proj, ldp, tail, tail_ld);
    if (!m->f32 && rows.prompt && latent_prompt_supported(a, n))
      check(m, r, launch_latent_prompt(a, l.w.up_map, rows, pos0, reinterpret_cast<bf16*>(out), ldo, m->c->status_word(), r.st, &r.launches), 0);
    else
      check(m, r, (launch_latent_rows<T, T, T>(a, rows, out, ldo, m->c->sm_count, false, r.st, &r.launches)), 0);
  } else {
    const DeltaArgs a = delta_args(m, l, run, proj, ldp, tail, tail_ld);
    if (rows.prompt) check(m, r, launch_delta_prompt<T>(a, rows, out, ldo, m->c->sm_count, r.st, &r.launches), 0);
    else check(m, r, (launch_delta_step<T, T>(a, rows, out, ldo, false, r.st)));
  }
}

// the gated half of a feed-forward: act(gate) * up of in -> h (ld ldh)
template <class T>
void ff_rows(Layered* m, LayeredRun& r, const LayerS& l, int n, const T* in, const XMaps& in_x, T* h, int64_t ldh) {
  const int ff = l.cfg.n_ff, act = l.cfg.ff_act == EMELB_FF_GELU_TANH ? ACT_GLU_GELU : ACT_GLU;
  const int64_t ldx = pad8(m->cfg.n_embd);
  if (m->f32) {
    linear(m, r, LinearArgs{l.w.ff_in, l.w.ff_in_bias, ACT_NONE, 0, n}, l.w.ff_in_map, in, ldx, in_x, m->gu, nullptr, 2 * ff);
    check(m, r, launch_glu_rows(m->gu, n, ff, act, reinterpret_cast<float*>(h), ldh, r.st));
  } else {
    linear(m, r, LinearArgs{l.w.ff_in, l.w.ff_in_bias, act, 0, n}, l.w.ff_in_map, in, ldx, in_x, nullptr, reinterpret_cast<bf16*>(h), ldh);
  }
}

template <class T>
void rows_through_layers(Layered* m, LayeredRun& r, const int* tokens, const Rows& rows, int pos0) {
  const int W = m->cfg.n_embd, n = rows.n;
  const int64_t ldx = pad8(W);
  T *xb = static_cast<T*>(m->xb), *xb2 = static_cast<T*>(m->xb2), *mix = static_cast<T*>(m->mix);
  const bool trace = m->trace_out && n <= m->trace_tokens;
  const size_t runs = m->runs.size();
  auto keep = [&](size_t i) { return trace ? m->trace_dev + (int64_t)i * n * W : nullptr; };
  // parallel layers: the sum behind run i - 1 and the norms in front of run i (i = runs: the sum alone)
  auto between = [&](size_t i) {
    PrenormArgs a{};
    a.x = m->x;
    if (i == 0) {
      a.table = m->embed.w;
      a.table_ld = m->embed.ld;
      a.tokens = tokens;
    } else {
      a.y = m->y;
      a.keep = keep(i - 1);
    }
    a.step = m->step_before(i);
    a.rms = m->rms();
    a.eps = m->cfg.rms_eps;
    a.rows = n;
    a.width = W;
    a.ldh = ldx;
    if (i < runs) {
      const LayerS& l = m->layers[m->runs[i].layer];
      a.w1 = l.w.norm1;
      a.h1 = xb;
      if (l.cfg.n_ff > 0) {
        a.w2 = l.w.norm2;
        a.h2 = xb2;
      }
    }
    check(m, r, launch_prenorm_rows<T>(a, r.st));
  };
  if (!m->parallel()) check(m, r, launch_embed_rows_bf16<T>(m->embed.w, m->embed.ld, tokens, m->step_before(0), n, W, m->x, xb, ldx, r.st));
  for (size_t i = 0; i < runs && r.ok; ++i) {
    const RunS& run = m->runs[i];
    const LayerS& l = m->layers[run.layer];
    const int ff = l.cfg.n_ff;
    if (m->parallel()) {
      between(i);
      if (ff > 0) {
        const int64_t ldj = pad8(l.joint_dim());
        mixer_rows<T>(m, r, l, run, rows, pos0, xb, m->xb_x, mix, ldj);
        ff_rows<T>(m, r, l, n, xb2, m->xb2_x, mix + pad8(l.out_dim()), ldj);
        linear(m, r, LinearArgs{l.w.out, l.w.ff_down_bias, ACT_NONE, 0, n}, l.w.out_map, mix, ldj, l.out_x, m->y, nullptr, W);
      } else {
        const int64_t ldo = pad8(l.out_dim());
        mixer_rows<T>(m, r, l, run, rows, pos0, xb, m->xb_x, mix, ldo);
        linear(m, r, LinearArgs{l.w.o, nullptr, ACT_NONE, 0, n}, l.w.o_map, mix, ldo, l.o_x, m->y, nullptr, W);
      }
      continue;
    }
    const int64_t ldo = pad8(l.out_dim());
    const float* next = m->step_before(i + 1);
    mixer_rows<T>(m, r, l, run, rows, pos0, xb, m->xb_x, mix, ldo);
    linear(m, r, LinearArgs{l.w.o, nullptr, ACT_NONE, 0, n}, l.w.o_map, mix, ldo, l.o_x, m->y, nullptr, W);
    check(m, r, launch_residual_norm<T>(m->x, m->y, l.w.norm1, m->rms(), m->cfg.rms_eps, n, W, xb, ldx, ff > 0 ? nullptr : keep(i), ff > 0 ? nullptr : next, r.st));
    if (ff > 0) {
      const int64_t ldh = pad8(ff);
      T* h = static_cast<T*>(m->h);
      ff_rows<T>(m, r, l, n, xb, m->xb_x, h, ldh);
      linear(m, r, LinearArgs{l.w.ff_down, l.w.ff_down_bias, ACT_NONE, 0, n}, l.w.ff_down_map, h, ldh, l.h_x, m->y, nullptr, W);
      check(m, r, launch_residual_norm<T>(m->x, m->y, l.w.norm2, m->rms(), m->cfg.rms_eps, n, W, xb, ldx, keep(i), next, r.st));
    }
  }
  if (m->parallel() && r.ok) between(runs);
  if (trace && r.ok)
    check(m, r, cudaMemcpyAsync(m->trace_out, m->trace_dev, 4 * runs * (size_t)n * W, cudaMemcpyDefault, r.st), 0);
}

// the fused one-token chain; T = type of the key / value cache
template <class T>
void step_through_layers(Layered* m, LayeredRun& r, int seq, const int* state, float* logits, int* argmax_parts) {
  const int sms = m->c->sm_count;
  const bool pdl = (m->c->pdl & 1) != 0;
  const Rows rows{1, false, seq, state + 1};
  int cur = 0;
  bool started = false;             // the stream is in vx[cur]
  const float* pending = nullptr;   // post-norm: norm of the sublayer output waiting in vy
  auto vec = [&](const Bf16Matrix& w, const float* bias, int act, int split, VecArgs v, float* out) {
    v.eps = m->cfg.rms_eps;
    v.rms = m->rms();
    v.out = out;
    LinearArgs a{w, bias, act, split, 1};
    if (act == ACT_SOFTCAP) {
      a.out_scale = m->stack.logit_scale;
      a.softcap = m->stack.logit_softcap;
    }
    check(m, r, launch_linear_vec(a, v, sms, pdl, r.st, v.part_val ? argmax_parts : nullptr));
  };
  // the stream as a product's prologue takes it: the table row, or the last stream and the output waiting in vy
  auto stream_in = [&](VecArgs& v, const float* step) {
    v.step = step;
    if (!started) {
      v.table = m->embed.w;
      v.table_ld = m->embed.ld;
      v.token = state;
    } else {
      v.x = m->vx[cur];
      v.y = m->vy;
      cur ^= 1;
    }
    v.x_out = m->vx[cur];
    started = true;
  };
  // post-norm: a product of the residual stream; the norm and sum of the sublayer before it run in its prologue
  auto stream = [&](const Bf16Matrix& w, const float* bias, int act, int split, const float* step, float* out) {
    VecArgs v{};
    v.pro = started ? PRO_RESIDUAL : PRO_EMBED;
    v.norm_w = pending;
    stream_in(v, step);
    vec(w, bias, act, split, v, out);
  };
  // a mixer's heads (or, where the output projection's prologue finishes them, what it needs: out) in vmix
  auto mixer = [&](const LayerS& l, const RunS& run, VecArgs& out) {
    if (l.attention()) {
      check(m, r, launch_attn_in<T>(attn_in_args(m, l, run, m->vproj, m->vq), rows, r.st));
      check(m, r, (launch_mix_attention_rows<T, float>(mix_args(m, l, run, m->vq), rows, m->vmix, l.out_dim(), sms, r.st, &r.launches)), 0);
    } else if (l.linear()) {
      check(m, r, launch_linear_attention_rows<float>(lin_args(m, l, run, 0, m->vmix), m->vproj, rows, r.st));
      out.pro = PRO_RMS_GATE;
      out.norm_w = l.w.norm_out;
      out.gate = m->vproj + l.linear_gate_at();
    } else if (l.latent()) {
      check(m, r, (launch_latent_rows<T, float, float>(latent_args(m, l, run, m->vproj, 0, m->vproj + l.tail_at(), 0), rows, m->vmix, 0, sms, pdl, r.st, &r.launches)), 0);
    } else {
      check(m, r, (launch_delta_step<float, float>(delta_args(m, l, run, m->vproj, 0, m->vproj + l.tail_at(), 0), rows, m->vmix, 0, pdl, r.st)));
    }
  };
  auto in_act = [](const LayerS& l) { return l.linear() ? ACT_SILU_SIGMOID : ACT_NONE; };
  auto ff_act = [](const LayerS& l) { return l.cfg.ff_act == EMELB_FF_GELU_TANH ? ACT_GLU_GELU : ACT_GLU; };
  for (size_t i = 0; i < m->runs.size() && r.ok; ++i) {
    const RunS& run = m->runs[i];
    const LayerS& l = m->layers[run.layer];
    const int split = l.linear() ? l.linear_gate_at() : 0;
    VecArgs out{};
    out.pro = PRO_PLAIN;
    out.x = m->vmix;
    if (m->parallel()) {
      // both inputs in one launch, both outputs in another
      VecArgs v{};
      v.pro = PRO_PRENORM;
      v.norm_w = l.w.norm1;
      stream_in(v, m->step_before(i));
      if (l.cfg.n_ff > 0) {
        v.norm2_w = l.w.norm2;
        v.w2 = l.w.ff_in;
        v.bias2 = l.w.ff_in_bias;
        v.act2 = ff_act(l);
        v.out2 = m->vmix + pad8(l.out_dim());
      }
      vec(l.w.in, nullptr, in_act(l), split, v, m->vproj);
      mixer(l, run, out);
      if (out.pro == PRO_RMS_GATE && l.cfg.n_ff > 0) {
        // the gated norm is of the heads alone, not of the joint vector
        check(m, r, launch_rms_gate<float>(m->vmix, l.w.norm_out, out.gate, l.in_rows, m->cfg.rms_eps, 1, l.out_dim(), m->vmix, l.out_dim(), r.st));
        out.pro = PRO_PLAIN;
      }
      if (l.cfg.n_ff > 0) vec(l.w.out, l.w.ff_down_bias, ACT_NONE, 0, out, m->vy);
      else vec(l.w.o, nullptr, ACT_NONE, 0, out, m->vy);
      continue;
    }
    stream(l.w.in, nullptr, in_act(l), split, m->step_before(i), m->vproj);
    mixer(l, run, out);
    vec(l.w.o, nullptr, ACT_NONE, 0, out, m->vy);
    pending = l.w.norm1;
    if (l.cfg.n_ff > 0) {
      stream(l.w.ff_in, l.w.ff_in_bias, ff_act(l), 0, nullptr, m->vh);
      VecArgs d{};
      d.pro = PRO_PLAIN;
      d.x = m->vh;
      vec(l.w.ff_down, l.w.ff_down_bias, ACT_NONE, 0, d, m->vy);
      pending = l.w.norm2;
    }
  }
  if (!logits || !r.ok) return;
  VecArgs v{};
  v.x = m->vx[cur];
  v.y = m->vy;
  if (m->parallel()) {
    v.pro = PRO_PRENORM;
    v.norm_w = m->final_norm;
  } else {
    v.pro = PRO_RESIDUAL_NORM;
    v.norm_w = pending;
    v.norm2_w = m->final_norm;
  }
  if (argmax_parts) {
    v.part_val = m->c->part_val;
    v.part_idx = m->c->part_idx;
  }
  vec(m->head, nullptr, ACT_SOFTCAP, 0, v, logits);
}

}  // namespace

emelb_stack_config layered_default_stack() {
  emelb_stack_config s{};
  s.arrangement = EMELB_STACK_POST_NORM;
  s.norm = EMELB_NORM_LAYER;
  s.logit_scale = 1.0f;
  return s;
}

uint32_t layered_check(const emelb_llama_config& c, const emelb_stack_config& st, const emelb_layer_config* layers) {
  if (!layers || c.n_layer < 1 || c.n_embd < 1 || c.n_vocab < 1 || c.n_ctx < 1 || c.shard_count > 1 || !(c.rms_eps >= 0.0f)) return EMELB_INVALID_REQUEST;
  if (c.n_embd > 40000) return EMELB_INVALID_REQUEST;   // a row's norm keeps it in shared memory
  const bool parallel = st.arrangement == EMELB_STACK_PARALLEL;
  if ((st.arrangement != EMELB_STACK_POST_NORM && !parallel) || (st.norm != EMELB_NORM_LAYER && st.norm != EMELB_NORM_RMS)) return EMELB_INVALID_REQUEST;
  if (parallel && c.n_embd > 20000) return EMELB_INVALID_REQUEST;   // both normed inputs
  if (st.loop_times < 0 || (st.loop_times > 0 && (st.loop_start < 0 || st.loop_stop <= st.loop_start || st.loop_stop > c.n_layer)) ||
      (st.loop_times == 0 && st.loop_step) || !std::isfinite(st.logit_scale) || !(st.logit_softcap >= 0.0f))
    return EMELB_INVALID_REQUEST;
  for (int i = 0; i < c.n_layer; ++i) {
    const emelb_layer_config& l = layers[i];
    if (l.n_head < 1 || l.key_dim < 1 || l.value_dim < 1 || l.n_ff < 0) return EMELB_INVALID_REQUEST;
    if (l.ff_act != EMELB_FF_SILU && l.ff_act != EMELB_FF_GELU_TANH) return EMELB_INVALID_REQUEST;
    // widths a product's or a norm's row may have (shared memory)
    if ((int64_t)l.n_head * l.value_dim > 40000 || (int64_t)l.n_head * l.key_dim > 40000 || l.n_ff > 50000) return EMELB_INVALID_REQUEST;
    if (parallel && (int64_t)l.n_head * l.value_dim + l.n_ff > 50000) return EMELB_INVALID_REQUEST;
    const bool rope_ok = l.rope_dim >= 0 && l.rope_dim % 2 == 0 && (l.rope_dim == 0 || l.rope_freq_base > 0.0f);
    if (l.mixer == EMELB_MIXER_LINEAR) {
      if (!l.decay || l.key_dim > 1024) return EMELB_INVALID_REQUEST;
    } else if (l.mixer == EMELB_MIXER_ATTENTION) {
      if (l.n_head_kv < 1 || l.n_head % l.n_head_kv != 0 || l.conv_taps < 0 || !rope_ok || l.rope_dim > l.key_dim ||
          l.window < 0 || l.keep_first < 0 || l.n_head > 256 || (int64_t)l.n_head_kv * l.value_dim > 40000)
        return EMELB_INVALID_REQUEST;
      if (l.kv_from >= i || l.kv_from < -1) return EMELB_INVALID_REQUEST;
      if (l.kv_from >= 0) {
        const emelb_layer_config& o = layers[l.kv_from];
        if (o.mixer != EMELB_MIXER_ATTENTION || o.kv_from >= 0 || o.n_head_kv != l.n_head_kv || o.key_dim != l.key_dim || o.value_dim != l.value_dim ||
            o.norm_v != l.norm_v)
          return EMELB_INVALID_REQUEST;
      }
    } else if (l.mixer == EMELB_MIXER_LATENT) {
      if (l.kv_rank < 1 || !rope_ok || l.window < 0 || (int64_t)l.n_head * (l.key_dim + l.rope_dim) > 40000 || l.kv_rank + l.rope_dim > 5000 ||
          l.key_dim > 8192)
        return EMELB_INVALID_REQUEST;
    } else if (l.mixer == EMELB_MIXER_DELTA) {
      if (l.n_head_kv < 1 || l.n_head % l.n_head_kv != 0 || l.conv_taps < 1 || l.key_dim > 1024 || l.value_dim > 8192 ||
          (int64_t)l.n_head_kv * l.key_dim > 40000)
        return EMELB_INVALID_REQUEST;
    } else {
      return EMELB_INVALID_REQUEST;
    }
  }
  return EMELB_OK;
}

Layered* layered_create(emelb_ctx* c, const emelb_llama_config& cfg, const emelb_stack_config& stack, const emelb_layer_config* layers, bool f32) {
  Layered* m = new (std::nothrow) Layered();
  if (!m) return nullptr;
  m->c = c;
  m->cfg = cfg;
  m->stack = stack;
  m->f32 = f32;
  const int kvb = cfg.kv_block > 0 ? cfg.kv_block : 16;
  m->capacity = ((int64_t)cfg.n_ctx + kvb - 1) / kvb * kvb;
  m->layers.resize(cfg.n_layer);
  bool ok = true;
  std::map<std::pair<int, float>, std::pair<const float*, const float*>> tables;
  int max_in = 0, max_out = 0, max_ff = 0, max_q = 0;
  uint64_t scores = 0, stats = 0, part = 0, lin_state = 0, qlat = 0;
  for (int i = 0; i < cfg.n_layer; ++i) {
    LayerS& l = m->layers[i];
    l.cfg = layers[i];
    l.cfg.decay = nullptr;
    if (!l.attention()) l.cfg.kv_from = -1;
    if (l.linear() || l.delta()) l.cfg.rope_dim = l.cfg.window = 0;
    l.in_rows = in_rows_of(l.cfg);
    max_in = std::max(max_in, l.in_rows);
    max_out = std::max(max_out, m->parallel() ? l.joint_dim() : l.out_dim());
    max_ff = std::max(max_ff, l.cfg.n_ff);
    if (l.linear()) {
      lin_state = std::max<uint64_t>(lin_state, (uint64_t)l.cfg.n_head * l.cfg.key_dim * l.cfg.value_dim);
      ok = ok && alloc_n(m->owned, &l.decay, l.cfg.n_head);
      ok = ok && ctx_cuda_ok(c, cudaMemcpy(l.decay, layers[i].decay, 4 * (size_t)l.cfg.n_head, cudaMemcpyHostToDevice));
    } else if (l.attention()) {
      max_q = std::max<int>(max_q, l.cfg.n_head * (int)pad8(l.cfg.key_dim));
      const uint64_t stride = (max_visible(m, l.cfg) + 3) & ~3;
      scores = std::max<uint64_t>(scores, l.cfg.n_head * stride);
      stats = std::max<uint64_t>(stats, 2ull * kMixAttnMaxSplits * l.cfg.n_head);
      part = std::max<uint64_t>(part, (uint64_t)kMixAttnMaxSplits * l.out_dim());
    } else if (l.latent()) {
      qlat = std::max<uint64_t>(qlat, (uint64_t)kLatentRows * l.cfg.n_head * l.cache_width());
      stats = std::max<uint64_t>(stats, 2ull * kMixAttnMaxSplits * kLatentRows * l.cfg.n_head);
      part = std::max<uint64_t>(part, (uint64_t)kMixAttnMaxSplits * l.cfg.n_head * l.rank_pad());
    }
    if (l.cfg.rope_dim > 0) {
      // cos / sin of position * base^(-2p / dims), from double angles
      auto& t = tables[{l.cfg.rope_dim, l.cfg.rope_freq_base}];
      if (!t.first) {
        const int pairs = l.cfg.rope_dim / 2;
        std::vector<float> hc((size_t)cfg.n_ctx * pairs), hs((size_t)cfg.n_ctx * pairs);
        for (int p = 0; p < pairs; ++p) {
          const double f = std::pow((double)l.cfg.rope_freq_base, -2.0 * p / l.cfg.rope_dim);
          for (int pos = 0; pos < cfg.n_ctx; ++pos) {
            hc[(size_t)pos * pairs + p] = (float)std::cos(pos * f);
            hs[(size_t)pos * pairs + p] = (float)std::sin(pos * f);
          }
        }
        float *dc = nullptr, *ds = nullptr;
        ok = ok && alloc_n(m->owned, &dc, hc.size()) && alloc_n(m->owned, &ds, hs.size());
        ok = ok && ctx_cuda_ok(c, cudaMemcpy(dc, hc.data(), 4 * hc.size(), cudaMemcpyHostToDevice)) &&
             ctx_cuda_ok(c, cudaMemcpy(ds, hs.data(), 4 * hs.size(), cudaMemcpyHostToDevice));
        t = {dc, ds};
      }
      l.rope_cos = t.first;
      l.rope_sin = t.second;
    }
  }
  // the order the layers run in
  const int times = stack.loop_times, start = times > 0 ? stack.loop_start : 0, stop = times > 0 ? stack.loop_stop : 0;
  auto add_run = [&](int layer, int pass) {
    RunS run;
    run.layer = layer;
    run.pass = pass;
    for (int i = (int)m->runs.size() - 1; i >= 0 && run.kv_run < 0; --i)
      if (m->runs[i].layer == m->layers[layer].cfg.kv_from) run.kv_run = i;   // the owner's latest
    m->runs.push_back(run);
  };
  for (int i = 0; i < start; ++i) add_run(i, -1);
  for (int t = 0; t < times; ++t)
    for (int i = start; i < stop; ++i) add_run(i, i == start ? t : -1);
  for (int i = stop; i < cfg.n_layer; ++i) add_run(i, -1);
  for (int i = 0; i < 2; ++i) ok = ok && alloc_n(m->owned, &m->vx[i], cfg.n_embd);
  ok = ok && alloc_n(m->owned, &m->vy, cfg.n_embd) && alloc_n(m->owned, &m->vproj, max_in) && alloc_n(m->owned, &m->vmix, max_out);
  if (ok) ok = ctx_cuda_ok(c, cudaMemset(m->vmix, 0, 4 * (size_t)max_out));   // padding inside the joint vector meets zeros: keep it finite
  if (max_ff > 0) ok = ok && alloc_n(m->owned, &m->vh, max_ff);
  if (lin_state > 0 && !f32) ok = ok && alloc_n(m->owned, &m->lin_local, kLinAttnMaxSegments * lin_state);
  if (scores > 0) {
    ok = ok && alloc(m->owned, &m->vq, 4 * (size_t)max_q);
    m->scores_floats = std::max<uint64_t>(scores, 16u << 20);
    // prompts keep one {max, sum} pair per 64 columns of a strip's scores
    stats = std::max<uint64_t>(stats, m->scores_floats / 32);
    ok = ok && alloc_n(m->owned, &m->scores, m->scores_floats);
  }
  if (part > 0) {
    m->stats_floats = stats;
    m->part_floats = std::max<uint64_t>(part, 4u << 20);
    ok = ok && alloc_n(m->owned, &m->stats, m->stats_floats) && alloc_n(m->owned, &m->part, m->part_floats);
  }
  if (qlat > 0) ok = ok && alloc_n(m->owned, &m->qlat, qlat);
  ok = ok && layered_set_sequences(m, 1);
  if (!ok) {
    layered_destroy(m);
    return nullptr;
  }
  return m;
}

void layered_destroy(Layered* m) {
  if (!m) return;
  free_all(m->owned);
  free_all(m->seq_owned);
  free_all(m->row_owned);
  delete m;
}

bool layered_set_sequences(Layered* m, int n_seq) {
  if (n_seq == m->n_seq) return true;
  if (cudaStreamSynchronize(m->c->stream) != cudaSuccess) {
    cudaGetLastError();
    return false;
  }
  free_all(m->seq_owned);
  m->n_seq = 0;
  bool ok = true;
  auto zeroed = [&](void** p, size_t bytes) {
    ok = ok && alloc(m->seq_owned, p, bytes) && ctx_cuda_ok(m->c, cudaMemsetAsync(*p, 0, bytes, m->c->stream));
  };
  for (RunS& run : m->runs) {
    const LayerS& l = m->layers[run.layer];
    const emelb_layer_config& g = l.cfg;
    run.k = run.v = nullptr;
    run.conv_state = run.state = nullptr;
    const size_t n = (size_t)n_seq;
    if (l.attention()) {
      if (l.own_kv()) {
        zeroed(&run.k, n * g.n_head_kv * m->capacity * pad8(g.key_dim) * m->operand_bytes());
        zeroed(&run.v, n * g.n_head_kv * m->capacity * pad8(g.value_dim) * m->operand_bytes());
      }
      if (g.conv_taps > 1) zeroed(reinterpret_cast<void**>(&run.conv_state), 4 * n * l.in_rows * (g.conv_taps - 1));
    } else if (l.latent()) {
      zeroed(&run.k, n * m->capacity * l.cache_width() * m->operand_bytes());
    } else {
      zeroed(reinterpret_cast<void**>(&run.state), 4 * n * g.n_head * (size_t)g.key_dim * g.value_dim);
      if (l.delta()) zeroed(reinterpret_cast<void**>(&run.conv_state), 4 * n * l.conv_channels() * (size_t)g.conv_taps);
    }
  }
  ok = ok && ctx_cuda_ok(m->c, cudaStreamSynchronize(m->c->stream));
  if (ok) m->n_seq = n_seq;
  return ok;
}

int layered_row_capacity(const Layered* m) { return m->row_cap; }

bool layered_reserve_rows(Layered* m, int rows) {
  if (m->row_cap >= rows) return true;
  if (cudaStreamSynchronize(m->c->stream) != cudaSuccess) {
    cudaGetLastError();
    return false;
  }
  free_all(m->row_owned);
  m->row_cap = 0;
  size_t in = 0, inb = 0, out = 0, lin = 0, ff = 0, q = 0, tail = 0, kv = 0, qkv = 0, scalars = 0, heads = 0;
  for (const LayerS& l : m->layers) {
    const emelb_layer_config& g = l.cfg;
    if (l.attention()) {
      in = std::max<size_t>(in, l.in_rows);
      q = std::max<size_t>(q, g.n_head * pad8(g.key_dim));
    } else {
      inb = std::max<size_t>(inb, pad8(l.in_rows));
      tail = std::max<size_t>(tail, l.in_rows - l.tail_at());
    }
    if (l.linear() || l.delta()) lin = std::max<size_t>(lin, l.out_dim());
    if (l.latent()) kv = std::max<size_t>(kv, std::min<size_t>(m->cfg.n_ctx, g.window > 0 ? (size_t)g.window + rows : m->cfg.n_ctx) * pad8(l.up_rows()));
    if (l.delta()) {
      qkv = std::max<size_t>(qkv, pad8(l.conv_channels()));
      scalars = std::max<size_t>(scalars, 2 * (g.n_head + g.n_head_kv));
      heads = std::max<size_t>(heads, g.n_head);
    }
    out = std::max<size_t>(out, pad8(m->parallel() ? l.joint_dim() : l.out_dim()));
    ff = std::max<size_t>(ff, g.n_ff);
  }
  const size_t n = rows, W = m->cfg.n_embd, ob = m->operand_bytes();
  bool ok = alloc_n(m->row_owned, &m->x, n * W) && alloc_n(m->row_owned, &m->y, n * W);
  ok = ok && alloc(m->row_owned, &m->xb, n * pad8(W) * ob) && alloc(m->row_owned, &m->nb, n * pad8(W) * ob);
  if (m->parallel()) ok = ok && alloc(m->row_owned, &m->xb2, n * pad8(W) * ob);
  if (in) ok = ok && alloc_n(m->row_owned, &m->proj, n * in) && alloc(m->row_owned, &m->q, n * q * ob);
  if (inb) ok = ok && alloc(m->row_owned, &m->projb, n * inb * ob);
  if (lin) ok = ok && alloc_n(m->row_owned, &m->lin, n * lin);
  if (tail && !m->f32) ok = ok && alloc_n(m->row_owned, &m->tail, n * tail);
  m->kv_elems = m->f32 ? 0 : kv;
  if (m->kv_elems) ok = ok && alloc_n(m->row_owned, &m->kv, kv);
  if (qkv) ok = ok && alloc(m->row_owned, &m->qkv, n * qkv * ob) && alloc_n(m->row_owned, &m->delta_scalars, n * scalars);
  if (qkv && !m->f32) ok = ok && alloc_n(m->row_owned, &m->delta_chunk, delta_chunk_floats() * delta_chunks(rows) * heads);
  ok = ok && alloc(m->row_owned, &m->mix, n * out * ob) && ctx_cuda_ok(m->c, cudaMemset(m->mix, 0, n * out * ob));
  if (ff && !m->parallel()) ok = ok && alloc(m->row_owned, &m->h, n * pad8(ff) * ob);
  if (ff && m->f32) ok = ok && alloc_n(m->row_owned, &m->gu, n * 2 * ff);
  if (ok && !m->f32) {
    ok = x_maps(&m->xb_x, m->xb, n, W, pad8(W)) && x_maps(&m->nb_x, m->nb, n, W, pad8(W));
    if (m->parallel()) ok = ok && x_maps(&m->xb2_x, m->xb2, n, W, pad8(W));
    for (LayerS& l : m->layers) {
      ok = ok && x_maps(&l.o_x, m->mix, n, l.out_dim(), pad8(l.out_dim()));
      if (m->parallel()) ok = ok && x_maps(&l.out_x, m->mix, n, l.joint_dim(), pad8(l.joint_dim()));
      else if (l.cfg.n_ff > 0) ok = ok && x_maps(&l.h_x, m->h, n, l.cfg.n_ff, pad8(l.cfg.n_ff));
    }
  }
  if (ok) m->row_cap = rows;
  return ok;
}

void layered_set_trace(Layered* m, float* out, int max_tokens) {
  m->trace_out = nullptr;
  if (!out || max_tokens < 1) return;
  if (max_tokens > m->trace_tokens || !m->trace_dev) {
    m->trace_dev = nullptr;   // the old buffer is freed with the model
    if (!alloc_n(m->owned, &m->trace_dev, m->runs.size() * (size_t)max_tokens * m->cfg.n_embd)) return;
    m->trace_tokens = max_tokens;
  }
  m->trace_out = out;
}

uint32_t layered_bind(Layered* m, int layer, int role, const emelb_view* t) {
  const emelb_llama_config& c = m->cfg;
  const bool model_level = (role >= EMELB_T_TOKEN_EMBD && role <= EMELB_T_OUTPUT) || role == EMELB_T_LOOP_STEP;
  if (!t || !t->data || (model_level ? layer != -1 : (layer < 0 || layer >= c.n_layer))) return EMELB_INVALID_REQUEST;
  LayerS* l = model_level ? nullptr : &m->layers[layer];
  Bf16Matrix* mat = nullptr;
  TmaMap* map = nullptr;
  const float** vec = nullptr;
  int64_t K = 0, M = 1;
  const bool att = l && l->attention(), ff = l && l->cfg.n_ff > 0, lat = l && l->latent(), del = l && l->delta();
  const bool joint = m->parallel() && ff;
  const emelb_layer_config* g = l ? &l->cfg : nullptr;
  switch (role) {
    case EMELB_T_TOKEN_EMBD: mat = &m->embed; K = c.n_embd; M = c.n_vocab; break;
    case EMELB_T_OUTPUT: mat = &m->head; map = &m->head_map; K = c.n_embd; M = c.n_vocab; break;
    case EMELB_T_OUTPUT_NORM: vec = &m->final_norm; K = c.n_embd; break;
    case EMELB_T_ATTN_NORM: vec = &l->w.norm1; K = c.n_embd; break;
    case EMELB_T_FFN_NORM: if (ff) { vec = &l->w.norm2; K = c.n_embd; } break;
    case EMELB_T_MIX_IN: mat = &l->w.in; map = &l->w.in_map; K = c.n_embd; M = l->in_rows; break;
    case EMELB_T_ATTN_OUT: if (!joint) { mat = &l->w.o; map = &l->w.o_map; K = l->out_dim(); M = c.n_embd; } break;
    case EMELB_T_LAYER_OUT: if (joint) { mat = &l->w.out; map = &l->w.out_map; K = l->joint_dim(); M = c.n_embd; } break;
    case EMELB_T_LOOP_STEP: if (m->stack.loop_step) { vec = &m->loop_step; K = c.n_embd; M = m->stack.loop_times; } break;
    case EMELB_T_MIX_LATENT_NORM: if (lat) { vec = &l->w.norm_latent; K = g->kv_rank; } break;
    case EMELB_T_MIX_LATENT_UP: if (lat) { mat = &l->w.up; map = &l->w.up_map; K = g->kv_rank; M = l->up_rows(); } break;
    case EMELB_T_MIX_DECAY_LOG: if (del) { vec = &l->w.decay_log; K = g->n_head; } break;
    case EMELB_T_MIX_STEP_BIAS: if (del) { vec = &l->w.step_bias; K = g->n_head; } break;
    case EMELB_T_MIX_CONV: if ((att || del) && g->conv_taps > 0) { vec = &l->w.conv; K = g->conv_taps; M = l->conv_channels(); } break;
    case EMELB_T_MIX_NORM_Q: if (att && g->norm_qk) { vec = &l->w.norm_q; K = (int64_t)g->n_head * g->key_dim; } break;
    case EMELB_T_MIX_NORM_K: if (att && g->norm_qk && l->own_kv()) { vec = &l->w.norm_k; K = (int64_t)g->n_head_kv * g->key_dim; } break;
    case EMELB_T_MIX_HEADS: if (att && g->mix_heads) { vec = &l->w.talk; K = M = g->n_head; } break;
    case EMELB_T_MIX_NORM_OUT: if (l->linear() || del) { vec = &l->w.norm_out; K = del ? g->value_dim : l->out_dim(); } break;
    case EMELB_T_FFN_IN: if (ff) { mat = &l->w.ff_in; map = &l->w.ff_in_map; K = c.n_embd; M = 2 * (int64_t)g->n_ff; } break;
    case EMELB_T_FFN_IN_BIAS: if (ff && g->ff_bias) { vec = &l->w.ff_in_bias; K = 2 * (int64_t)g->n_ff; } break;
    case EMELB_T_FFN_DOWN: if (ff && !joint) { mat = &l->w.ff_down; map = &l->w.ff_down_map; K = g->n_ff; M = c.n_embd; } break;
    case EMELB_T_FFN_DOWN_BIAS: if (ff && g->ff_bias) { vec = &l->w.ff_down_bias; K = c.n_embd; } break;
    default: break;
  }
  if (!mat && !vec) return EMELB_INVALID_REQUEST;
  if ((int64_t)t->ne[0] != K || (int64_t)t->ne[1] != M) return EMELB_INVALID_REQUEST;
  const void* dev = ctx_resolve_weights(m->c, t->data);
  if (!dev) return EMELB_INVALID_REQUEST;
  if (vec) {
    if (t->type != EMELB_F32 || t->nb[0] != 4 || (M > 1 && (int64_t)t->nb[1] != 4 * K) || reinterpret_cast<uintptr_t>(dev) % 16 != 0) return EMELB_INVALID_REQUEST;
    if (role == EMELB_T_MIX_CONV) {
      // kept tap by tap, so that neighbouring channels are read together
      float* taps = const_cast<float*>(l->w.conv);
      if (!taps && !alloc_n(m->owned, &taps, (size_t)(K * M))) return EMELB_INTERNAL_ERROR;
      if (!ctx_cuda_ok(m->c, launch_transpose(static_cast<const float*>(dev), (int)M, (int)K, taps, m->c->stream))) return EMELB_INTERNAL_ERROR;
      dev = taps;
    }
    *vec = static_cast<const float*>(dev);
    return EMELB_OK;
  }
  if (t->type != EMELB_BF16 || t->nb[0] != 2 || t->nb[1] % 16 != 0 || (int64_t)t->nb[1] < 2 * K || reinterpret_cast<uintptr_t>(dev) % 16 != 0)
    return EMELB_INVALID_REQUEST;
  Bf16Matrix w;
  w.w = static_cast<const bf16*>(dev);
  w.ld = (int64_t)t->nb[1] / 2;
  w.M = (int)M;
  w.K = (int)K;
  if (map && !m->f32 && !encode_bf16_map(map, w.w, M, K, w.ld, kGemmWeightBox)) return EMELB_INTERNAL_ERROR;
  *mat = w;
  return EMELB_OK;
}

bool layered_bound(const Layered* m) {
  bool ok = m->embed.w && m->head.w && m->final_norm && (!m->stack.loop_step || m->loop_step);
  for (const LayerS& l : m->layers) {
    const emelb_layer_config& g = l.cfg;
    const bool ff = g.n_ff > 0, joint = m->parallel() && ff;
    ok = ok && l.w.in.w && (joint ? l.w.out.w : l.w.o.w) && l.w.norm1;
    if (l.attention()) {
      ok = ok && (g.conv_taps == 0 || l.w.conv) && (!g.norm_qk || (l.w.norm_q && (!l.own_kv() || l.w.norm_k))) && (!g.mix_heads || l.w.talk);
    } else if (l.latent()) {
      ok = ok && l.w.norm_latent && l.w.up.w;
    } else {
      ok = ok && l.w.norm_out;
      if (l.delta()) ok = ok && l.w.conv && l.w.decay_log && l.w.step_bias;
    }
    if (ff) ok = ok && l.w.norm2 && l.w.ff_in.w && (joint || l.w.ff_down.w) && (!g.ff_bias || (l.w.ff_in_bias && l.w.ff_down_bias));
  }
  return ok;
}

void layered_step(Layered* m, LayeredRun& r, int seq, const int* state, float* logits, int* argmax_parts) {
  if (m->f32) step_through_layers<float>(m, r, seq, state, logits, argmax_parts);
  else step_through_layers<bf16>(m, r, seq, state, logits, argmax_parts);
}

void layered_rows(Layered* m, LayeredRun& r, const int* tokens, const Rows& rows, int pos0) {
  if (m->f32) rows_through_layers<float>(m, r, tokens, rows, pos0);
  else rows_through_layers<bf16>(m, r, tokens, rows, pos0);
}

void layered_rows_logits(Layered* m, LayeredRun& r, const int* index, int n, float* logits) {
  const int W = m->cfg.n_embd;
  const int64_t ld = pad8(W);
  if (m->f32) check(m, r, launch_norm_rows<float>(m->x, index, m->final_norm, m->rms(), m->cfg.rms_eps, n, W, static_cast<float*>(m->nb), ld, r.st));
  else check(m, r, launch_norm_rows<bf16>(m->x, index, m->final_norm, m->rms(), m->cfg.rms_eps, n, W, static_cast<bf16*>(m->nb), ld, r.st));
  LinearArgs a{m->head, nullptr, ACT_SOFTCAP, 0, n};
  a.out_scale = m->stack.logit_scale;
  a.softcap = m->stack.logit_softcap;
  linear(m, r, a, m->head_map, m->nb, ld, m->nb_x, logits, nullptr, m->cfg.n_vocab);
}

}  // namespace emelb
