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
  Bf16Matrix in, o, ff_in, ff_down;
  TmaMap in_map, o_map, ff_in_map, ff_down_map;
  const float *conv = nullptr, *norm_q = nullptr, *norm_k = nullptr, *talk = nullptr, *norm_out = nullptr;
  const float *norm1 = nullptr, *norm2 = nullptr, *ff_in_bias = nullptr, *ff_down_bias = nullptr;
};

struct LayerS {
  emelb_layer_config cfg{};
  int in_rows = 0;              // rows of the stacked input projections
  float* decay = nullptr;       // linear
  const float *rope_cos = nullptr, *rope_sin = nullptr;
  // per sequence
  void *k = nullptr, *v = nullptr;
  float* conv_state = nullptr;
  float* state = nullptr;
  LayerW w;
  XMaps o_x{}, h_x{};           // the operand buffers as this layer's products read them
  bool own_kv() const { return cfg.kv_from < 0; }
  bool attention() const { return cfg.mixer == EMELB_MIXER_ATTENTION; }
  int out_dim() const { return cfg.n_head * cfg.value_dim; }
  int gate_at() const { return 2 * cfg.n_head * cfg.key_dim + cfg.n_head * cfg.value_dim; }
};

int in_rows_of(const emelb_layer_config& l) {
  if (l.mixer == EMELB_MIXER_LINEAR) return 2 * l.n_head * l.key_dim + 2 * l.n_head * l.value_dim;
  return l.n_head * l.key_dim + (l.kv_from < 0 ? l.n_head_kv * (l.key_dim + l.value_dim) : 0);
}

}  // namespace

struct Layered {
  emelb_ctx* c = nullptr;
  emelb_llama_config cfg{};
  bool f32 = false;
  std::vector<LayerS> layers;
  Bf16Matrix embed, head;
  TmaMap head_map;
  const float* final_norm = nullptr;
  int64_t capacity = 0;
  int n_seq = 0;
  std::vector<void*> owned, seq_owned, row_owned;
  // one token
  float *vx[2] = {nullptr, nullptr}, *vproj = nullptr, *vmix = nullptr, *vh = nullptr, *vy = nullptr;
  void* vq = nullptr;
  // rows
  int row_cap = 0;
  float *x = nullptr, *y = nullptr, *proj = nullptr, *lin = nullptr, *gu = nullptr;
  void *xb = nullptr, *projb = nullptr, *q = nullptr, *mix = nullptr, *h = nullptr, *nb = nullptr;
  XMaps xb_x{}, nb_x{};
  // attention scratch
  float* lin_local = nullptr;
  float *scores = nullptr, *stats = nullptr, *part = nullptr;
  uint64_t scores_floats = 0, stats_floats = 0, part_floats = 0;
  float* trace_out = nullptr;
  float* trace_dev = nullptr;
  int trace_tokens = 0;

  size_t operand_bytes() const { return f32 ? 4 : 2; }
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

AttnInArgs attn_in_args(const Layered* m, const LayerS& l, const float* proj, void* q) {
  const emelb_layer_config& g = l.cfg;
  AttnInArgs a{};
  a.proj = proj;
  a.channels = l.in_rows;
  a.conv = l.w.conv;
  a.taps = g.conv_taps > 0 ? g.conv_taps : 1;
  a.conv_state = l.conv_state;
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
  a.k = l.k;
  a.v = l.v;
  a.capacity = m->capacity;
  return a;
}

MixAttnArgs mix_args(const Layered* m, const LayerS& l, const void* q) {
  const emelb_layer_config& g = l.cfg;
  const LayerS& kv = l.own_kv() ? l : m->layers[g.kv_from];
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

LinAttnArgs lin_args(const Layered* m, const LayerS& l, int64_t ldx, float* out) {
  const emelb_layer_config& g = l.cfg;
  return LinAttnArgs{ldx, g.n_head, g.key_dim, g.value_dim, l.decay, l.state, out, m->lin_local};
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
void linear(Layered* m, LayeredRun& r, const Bf16Matrix& w, const TmaMap& wmap, const void* x, int64_t ldx, const XMaps& xm, int rows,
            const float* bias, int act, int split, float* y, bf16* yb, int64_t ldy) {
  LinearArgs a{w, bias, act, split, rows};
  if (m->f32) check(m, r, launch_linear_f32(a, static_cast<const float*>(x), ldx, y, ldy, r.st));
  else check(m, r, launch_gemm_bf16(a, wmap, xm, y, yb, ldy, m->c->status_word(), r.st));
}

template <class T>
void rows_through_layers(Layered* m, LayeredRun& r, const int* tokens, const Rows& rows, int pos0) {
  const int W = m->cfg.n_embd, n = rows.n;
  const int64_t ldx = pad8(W);
  T* xb = static_cast<T*>(m->xb);
  const bool trace = m->trace_out && n <= m->trace_tokens;
  check(m, r, launch_embed_rows_bf16<T>(m->embed.w, m->embed.ld, tokens, n, W, m->x, xb, ldx, r.st));
  for (size_t li = 0; li < m->layers.size() && r.ok; ++li) {
    LayerS& l = m->layers[li];
    const emelb_layer_config& g = l.cfg;
    const int od = l.out_dim();
    const int64_t ldo = pad8(od);
    T* mix = static_cast<T*>(m->mix);
    float* keep = trace ? m->trace_dev + (int64_t)li * n * W : nullptr;
    if (l.attention()) {
      linear(m, r, l.w.in, l.w.in_map, xb, ldx, m->xb_x, n, nullptr, ACT_NONE, 0, m->proj, nullptr, l.in_rows);
      const AttnInArgs in = attn_in_args(m, l, m->proj, m->q);
      check(m, r, launch_attn_in<T>(in, rows, r.st));
      if (rows.prompt && in.conv && in.taps > 1) check(m, r, launch_conv_state(in, rows, r.st));
      const MixAttnArgs a = mix_args(m, l, m->q);
      if (!m->f32 && rows.prompt && mix_attention_prompt_supported(a))
        check(m, r, launch_mix_attention_prompt(a, rows, pos0, reinterpret_cast<bf16*>(mix), ldo, r.st, &r.launches), 0);
      else
        check(m, r, (launch_mix_attention_rows<T, T>(a, rows, mix, ldo, m->c->sm_count, r.st, &r.launches)), 0);
    } else {
      const int64_t ldp = pad8(l.in_rows);
      T* proj = static_cast<T*>(m->projb);
      linear(m, r, l.w.in, l.w.in_map, xb, ldx, m->xb_x, n, nullptr, ACT_SILU_SIGMOID, l.gate_at(), reinterpret_cast<float*>(m->projb),
             m->f32 ? nullptr : static_cast<bf16*>(m->projb), ldp);
      const LinAttnArgs a = lin_args(m, l, ldp, m->lin);
      if (!m->f32 && rows.prompt && linear_attention_prompt_supported(a))
        check(m, r, launch_linear_attention_prompt(a, reinterpret_cast<const bf16*>(proj), rows, m->c->sm_count, r.st, &r.launches), 0);
      else
        check(m, r, launch_linear_attention_rows<T>(a, proj, rows, r.st));
      check(m, r, launch_rms_gate<T>(m->lin, l.w.norm_out, proj + l.gate_at(), ldp, m->cfg.rms_eps, n, od, mix, ldo, r.st));
    }
    linear(m, r, l.w.o, l.w.o_map, mix, ldo, l.o_x, n, nullptr, ACT_NONE, 0, m->y, nullptr, W);
    check(m, r, launch_residual_norm<T>(m->x, m->y, l.w.norm1, m->cfg.rms_eps, n, W, xb, ldx, g.n_ff > 0 ? nullptr : keep, r.st));
    if (g.n_ff > 0) {
      const int64_t ldh = pad8(g.n_ff);
      if (m->f32) {
        linear(m, r, l.w.ff_in, l.w.ff_in_map, xb, ldx, m->xb_x, n, l.w.ff_in_bias, ACT_NONE, 0, m->gu, nullptr, 2 * g.n_ff);
        check(m, r, launch_glu_rows(m->gu, n, g.n_ff, static_cast<float*>(m->h), ldh, r.st));
      } else {
        linear(m, r, l.w.ff_in, l.w.ff_in_map, xb, ldx, m->xb_x, n, l.w.ff_in_bias, ACT_GLU, 0, nullptr, static_cast<bf16*>(m->h), ldh);
      }
      linear(m, r, l.w.ff_down, l.w.ff_down_map, m->h, ldh, l.h_x, n, l.w.ff_down_bias, ACT_NONE, 0, m->y, nullptr, W);
      check(m, r, launch_residual_norm<T>(m->x, m->y, l.w.norm2, m->cfg.rms_eps, n, W, xb, ldx, keep, r.st));
    }
  }
  if (trace && r.ok)
    check(m, r, cudaMemcpyAsync(m->trace_out, m->trace_dev, 4 * m->layers.size() * (size_t)n * W, cudaMemcpyDefault, r.st), 0);
}

// the fused one-token chain; T = type of the key / value cache
template <class T>
void step_through_layers(Layered* m, LayeredRun& r, int seq, const int* state, float* logits, int* argmax_parts) {
  const int sms = m->c->sm_count;
  const bool pdl = (m->c->pdl & 1) != 0;
  const Rows rows{1, false, seq, state + 1};
  int cur = 0;
  const float* pending = nullptr;   // norm of the sublayer output waiting in vy
  auto vec = [&](const Bf16Matrix& w, const float* bias, int act, int split, VecArgs v, float* out) {
    v.eps = m->cfg.rms_eps;
    v.out = out;
    check(m, r, launch_linear_vec(LinearArgs{w, bias, act, split, 1}, v, sms, pdl, r.st, v.part_val ? argmax_parts : nullptr));
  };
  // a product of the residual stream: the norm and sum of the sublayer before it run in its prologue
  auto stream = [&](const Bf16Matrix& w, const float* bias, int act, int split, float* out) {
    VecArgs v{};
    if (!pending) {
      v.pro = PRO_EMBED;
      v.table = m->embed.w;
      v.table_ld = m->embed.ld;
      v.token = state;
      v.x_out = m->vx[cur];
    } else {
      v.pro = PRO_RESIDUAL;
      v.x = m->vx[cur];
      v.y = m->vy;
      v.norm_w = pending;
      cur ^= 1;
      v.x_out = m->vx[cur];
    }
    vec(w, bias, act, split, v, out);
  };
  for (size_t li = 0; li < m->layers.size() && r.ok; ++li) {
    LayerS& l = m->layers[li];
    const emelb_layer_config& g = l.cfg;
    VecArgs out{};
    out.pro = PRO_PLAIN;
    out.x = m->vmix;
    if (l.attention()) {
      stream(l.w.in, nullptr, ACT_NONE, 0, m->vproj);
      check(m, r, launch_attn_in<T>(attn_in_args(m, l, m->vproj, m->vq), rows, r.st));
      check(m, r, (launch_mix_attention_rows<T, float>(mix_args(m, l, m->vq), rows, m->vmix, l.out_dim(), sms, r.st, &r.launches)), 0);
    } else {
      stream(l.w.in, nullptr, ACT_SILU_SIGMOID, l.gate_at(), m->vproj);
      check(m, r, launch_linear_attention_rows<float>(lin_args(m, l, 0, m->vmix), m->vproj, rows, r.st));
      out.pro = PRO_RMS_GATE;
      out.norm_w = l.w.norm_out;
      out.gate = m->vproj + l.gate_at();
    }
    vec(l.w.o, nullptr, ACT_NONE, 0, out, m->vy);
    pending = l.w.norm1;
    if (g.n_ff > 0) {
      stream(l.w.ff_in, l.w.ff_in_bias, ACT_GLU, 0, m->vh);
      VecArgs d{};
      d.pro = PRO_PLAIN;
      d.x = m->vh;
      vec(l.w.ff_down, l.w.ff_down_bias, ACT_NONE, 0, d, m->vy);
      pending = l.w.norm2;
    }
  }
  if (!logits || !r.ok) return;
  VecArgs v{};
  v.pro = PRO_RESIDUAL_NORM;
  v.x = m->vx[cur];
  v.y = m->vy;
  v.norm_w = pending;
  v.norm2_w = m->final_norm;
  if (argmax_parts) {
    v.part_val = m->c->part_val;
    v.part_idx = m->c->part_idx;
  }
  vec(m->head, nullptr, ACT_NONE, 0, v, logits);
}

}  // namespace

uint32_t layered_check(const emelb_llama_config& c, const emelb_layer_config* layers) {
  if (!layers || c.n_layer < 1 || c.n_embd < 1 || c.n_vocab < 1 || c.n_ctx < 1 || c.shard_count > 1 || !(c.rms_eps >= 0.0f)) return EMELB_INVALID_REQUEST;
  if (c.n_embd > 40000) return EMELB_INVALID_REQUEST;   // a row's norm keeps it in shared memory
  for (int i = 0; i < c.n_layer; ++i) {
    const emelb_layer_config& l = layers[i];
    if (l.n_head < 1 || l.key_dim < 1 || l.value_dim < 1 || l.n_ff < 0) return EMELB_INVALID_REQUEST;
    // widths a product's or a norm's row may have (shared memory)
    if ((int64_t)l.n_head * l.value_dim > 40000 || (int64_t)l.n_head * l.key_dim > 40000 || l.n_ff > 50000) return EMELB_INVALID_REQUEST;
    if (l.mixer == EMELB_MIXER_LINEAR) {
      if (!l.decay || l.key_dim > 1024) return EMELB_INVALID_REQUEST;
    } else if (l.mixer == EMELB_MIXER_ATTENTION) {
      if (l.n_head_kv < 1 || l.n_head % l.n_head_kv != 0 || l.conv_taps < 0 || l.rope_dim < 0 || l.rope_dim % 2 != 0 || l.rope_dim > l.key_dim ||
          l.window < 0 || l.keep_first < 0 || l.n_head > 256 || (int64_t)l.n_head_kv * l.value_dim > 40000 ||
          (l.rope_dim > 0 && !(l.rope_freq_base > 0.0f)))
        return EMELB_INVALID_REQUEST;
      if (l.kv_from >= i || l.kv_from < -1) return EMELB_INVALID_REQUEST;
      if (l.kv_from >= 0) {
        const emelb_layer_config& o = layers[l.kv_from];
        if (o.mixer != EMELB_MIXER_ATTENTION || o.kv_from >= 0 || o.n_head_kv != l.n_head_kv || o.key_dim != l.key_dim || o.value_dim != l.value_dim ||
            o.norm_v != l.norm_v)
          return EMELB_INVALID_REQUEST;
      }
    } else {
      return EMELB_INVALID_REQUEST;
    }
  }
  return EMELB_OK;
}

Layered* layered_create(emelb_ctx* c, const emelb_llama_config& cfg, const emelb_layer_config* layers, bool f32) {
  Layered* m = new (std::nothrow) Layered();
  if (!m) return nullptr;
  m->c = c;
  m->cfg = cfg;
  m->f32 = f32;
  const int kvb = cfg.kv_block > 0 ? cfg.kv_block : 16;
  m->capacity = ((int64_t)cfg.n_ctx + kvb - 1) / kvb * kvb;
  m->layers.resize(cfg.n_layer);
  bool ok = true;
  std::map<std::pair<int, float>, std::pair<const float*, const float*>> tables;
  int max_in = 0, max_out = 0, max_ff = 0, max_q = 0;
  uint64_t scores = 0, stats = 0, part = 0, lin_state = 0;
  for (int i = 0; i < cfg.n_layer; ++i) {
    LayerS& l = m->layers[i];
    l.cfg = layers[i];
    l.cfg.decay = nullptr;
    if (!l.attention()) l.cfg.kv_from = -1;
    l.in_rows = in_rows_of(l.cfg);
    max_in = std::max(max_in, l.in_rows);
    max_out = std::max(max_out, l.out_dim());
    max_ff = std::max(max_ff, l.cfg.n_ff);
    if (!l.attention()) {
      lin_state = std::max<uint64_t>(lin_state, (uint64_t)l.cfg.n_head * l.cfg.key_dim * l.cfg.value_dim);
      ok = ok && alloc_n(m->owned, &l.decay, l.cfg.n_head);
      ok = ok && ctx_cuda_ok(c, cudaMemcpy(l.decay, layers[i].decay, 4 * (size_t)l.cfg.n_head, cudaMemcpyHostToDevice));
      continue;
    }
    max_q = std::max<int>(max_q, l.cfg.n_head * (int)pad8(l.cfg.key_dim));
    const uint64_t stride = (max_visible(m, l.cfg) + 3) & ~3;
    scores = std::max<uint64_t>(scores, l.cfg.n_head * stride);
    stats = std::max<uint64_t>(stats, 2ull * kMixAttnMaxSplits * l.cfg.n_head);
    part = std::max<uint64_t>(part, (uint64_t)kMixAttnMaxSplits * l.out_dim());
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
  for (int i = 0; i < 2; ++i) ok = ok && alloc_n(m->owned, &m->vx[i], cfg.n_embd);
  ok = ok && alloc_n(m->owned, &m->vy, cfg.n_embd) && alloc_n(m->owned, &m->vproj, max_in) && alloc_n(m->owned, &m->vmix, max_out);
  if (max_ff > 0) ok = ok && alloc_n(m->owned, &m->vh, max_ff);
  if (lin_state > 0 && !f32) ok = ok && alloc_n(m->owned, &m->lin_local, kLinAttnMaxSegments * lin_state);
  if (scores > 0) {
    ok = ok && alloc(m->owned, &m->vq, 4 * (size_t)max_q);
    m->scores_floats = std::max<uint64_t>(scores, 16u << 20);
    // prompts keep one {max, sum} pair per 64 columns of a strip's scores
    m->stats_floats = std::max<uint64_t>(stats, m->scores_floats / 32);
    m->part_floats = std::max<uint64_t>(part, 4u << 20);
    ok = ok && alloc_n(m->owned, &m->scores, m->scores_floats) && alloc_n(m->owned, &m->stats, m->stats_floats) &&
         alloc_n(m->owned, &m->part, m->part_floats);
  }
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
  for (LayerS& l : m->layers) {
    const emelb_layer_config& g = l.cfg;
    l.k = l.v = nullptr;
    l.conv_state = l.state = nullptr;
    const size_t n = (size_t)n_seq;
    if (l.attention()) {
      if (l.own_kv()) {
        zeroed(&l.k, n * g.n_head_kv * m->capacity * pad8(g.key_dim) * m->operand_bytes());
        zeroed(&l.v, n * g.n_head_kv * m->capacity * pad8(g.value_dim) * m->operand_bytes());
      }
      if (g.conv_taps > 1) zeroed(reinterpret_cast<void**>(&l.conv_state), 4 * n * l.in_rows * (g.conv_taps - 1));
    } else {
      zeroed(reinterpret_cast<void**>(&l.state), 4 * n * g.n_head * (size_t)g.key_dim * g.value_dim);
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
  size_t in = 0, inb = 0, out = 0, lin = 0, ff = 0, q = 0;
  for (const LayerS& l : m->layers) {
    if (l.attention()) {
      in = std::max<size_t>(in, l.in_rows);
      q = std::max<size_t>(q, l.cfg.n_head * pad8(l.cfg.key_dim));
    } else {
      inb = std::max<size_t>(inb, pad8(l.in_rows));
      lin = std::max<size_t>(lin, l.out_dim());
    }
    out = std::max<size_t>(out, pad8(l.out_dim()));
    ff = std::max<size_t>(ff, l.cfg.n_ff);
  }
  const size_t n = rows, W = m->cfg.n_embd, ob = m->operand_bytes();
  bool ok = alloc_n(m->row_owned, &m->x, n * W) && alloc_n(m->row_owned, &m->y, n * W);
  ok = ok && alloc(m->row_owned, &m->xb, n * pad8(W) * ob) && alloc(m->row_owned, &m->nb, n * pad8(W) * ob);
  if (in) ok = ok && alloc_n(m->row_owned, &m->proj, n * in) && alloc(m->row_owned, &m->q, n * q * ob);
  if (inb) ok = ok && alloc(m->row_owned, &m->projb, n * inb * ob) && alloc_n(m->row_owned, &m->lin, n * lin);
  ok = ok && alloc(m->row_owned, &m->mix, n * out * ob);
  if (ff) ok = ok && alloc(m->row_owned, &m->h, n * pad8(ff) * ob);
  if (ff && m->f32) ok = ok && alloc_n(m->row_owned, &m->gu, n * 2 * ff);
  if (ok && !m->f32) {
    ok = x_maps(&m->xb_x, m->xb, n, W, pad8(W)) && x_maps(&m->nb_x, m->nb, n, W, pad8(W));
    for (LayerS& l : m->layers) {
      ok = ok && x_maps(&l.o_x, m->mix, n, l.out_dim(), pad8(l.out_dim()));
      if (l.cfg.n_ff > 0) ok = ok && x_maps(&l.h_x, m->h, n, l.cfg.n_ff, pad8(l.cfg.n_ff));
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
    if (!alloc_n(m->owned, &m->trace_dev, m->layers.size() * (size_t)max_tokens * m->cfg.n_embd)) return;
    m->trace_tokens = max_tokens;
  }
  m->trace_out = out;
}

uint32_t layered_bind(Layered* m, int layer, int role, const emelb_view* t) {
  const emelb_llama_config& c = m->cfg;
  const bool model_level = role >= EMELB_T_TOKEN_EMBD && role <= EMELB_T_OUTPUT;
  if (!t || !t->data || (model_level ? layer != -1 : (layer < 0 || layer >= c.n_layer))) return EMELB_INVALID_REQUEST;
  LayerS* l = model_level ? nullptr : &m->layers[layer];
  Bf16Matrix* mat = nullptr;
  TmaMap* map = nullptr;
  const float** vec = nullptr;
  int64_t K = 0, M = 1;
  const bool att = l && l->attention(), ff = l && l->cfg.n_ff > 0;
  const emelb_layer_config* g = l ? &l->cfg : nullptr;
  switch (role) {
    case EMELB_T_TOKEN_EMBD: mat = &m->embed; K = c.n_embd; M = c.n_vocab; break;
    case EMELB_T_OUTPUT: mat = &m->head; map = &m->head_map; K = c.n_embd; M = c.n_vocab; break;
    case EMELB_T_OUTPUT_NORM: vec = &m->final_norm; K = c.n_embd; break;
    case EMELB_T_ATTN_NORM: vec = &l->w.norm1; K = c.n_embd; break;
    case EMELB_T_FFN_NORM: if (ff) { vec = &l->w.norm2; K = c.n_embd; } break;
    case EMELB_T_MIX_IN: mat = &l->w.in; map = &l->w.in_map; K = c.n_embd; M = l->in_rows; break;
    case EMELB_T_ATTN_OUT: mat = &l->w.o; map = &l->w.o_map; K = l->out_dim(); M = c.n_embd; break;
    case EMELB_T_MIX_CONV: if (att && g->conv_taps > 0) { vec = &l->w.conv; K = g->conv_taps; M = l->in_rows; } break;
    case EMELB_T_MIX_NORM_Q: if (att && g->norm_qk) { vec = &l->w.norm_q; K = (int64_t)g->n_head * g->key_dim; } break;
    case EMELB_T_MIX_NORM_K: if (att && g->norm_qk && l->own_kv()) { vec = &l->w.norm_k; K = (int64_t)g->n_head_kv * g->key_dim; } break;
    case EMELB_T_MIX_HEADS: if (att && g->mix_heads) { vec = &l->w.talk; K = M = g->n_head; } break;
    case EMELB_T_MIX_NORM_OUT: if (!att) { vec = &l->w.norm_out; K = l->out_dim(); } break;
    case EMELB_T_FFN_IN: if (ff) { mat = &l->w.ff_in; map = &l->w.ff_in_map; K = c.n_embd; M = 2 * (int64_t)g->n_ff; } break;
    case EMELB_T_FFN_IN_BIAS: if (ff) { vec = &l->w.ff_in_bias; K = 2 * (int64_t)g->n_ff; } break;
    case EMELB_T_FFN_DOWN: if (ff) { mat = &l->w.ff_down; map = &l->w.ff_down_map; K = g->n_ff; M = c.n_embd; } break;
    case EMELB_T_FFN_DOWN_BIAS: if (ff) { vec = &l->w.ff_down_bias; K = c.n_embd; } break;
    default: break;
  }
  if (!mat && !vec) return EMELB_INVALID_REQUEST;
  if ((int64_t)t->ne[0] != K || (int64_t)t->ne[1] != M) return EMELB_INVALID_REQUEST;
  const void* dev = ctx_resolve_weights(m->c, t->data);
  if (!dev) return EMELB_INVALID_REQUEST;
  if (vec) {
    if (t->type != EMELB_F32 || t->nb[0] != 4 || (M > 1 && (int64_t)t->nb[1] != 4 * K)) return EMELB_INVALID_REQUEST;
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
  bool ok = m->embed.w && m->head.w && m->final_norm;
  for (const LayerS& l : m->layers) {
    const emelb_layer_config& g = l.cfg;
    ok = ok && l.w.in.w && l.w.o.w && l.w.norm1;
    if (l.attention()) {
      ok = ok && (g.conv_taps == 0 || l.w.conv) && (!g.norm_qk || (l.w.norm_q && (!l.own_kv() || l.w.norm_k))) && (!g.mix_heads || l.w.talk);
    } else {
      ok = ok && l.w.norm_out;
    }
    if (g.n_ff > 0) ok = ok && l.w.norm2 && l.w.ff_in.w && l.w.ff_in_bias && l.w.ff_down.w && l.w.ff_down_bias;
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
  if (m->f32) check(m, r, launch_norm_rows<float>(m->x, index, m->final_norm, m->cfg.rms_eps, n, W, static_cast<float*>(m->nb), ld, r.st));
  else check(m, r, launch_norm_rows<bf16>(m->x, index, m->final_norm, m->cfg.rms_eps, n, W, static_cast<bf16*>(m->nb), ld, r.st));
  linear(m, r, m->head, m->head_map, m->nb, ld, m->nb_x, n, nullptr, ACT_NONE, 0, logits, nullptr, m->cfg.n_vocab);
}

}  // namespace emelb
