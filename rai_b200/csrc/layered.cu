// Decoders described layer by layer: every layer has its own sequence mixer (windowed attention or the HGRN2 recurrence),
// its own sizes and an optional feed-forward, with the norm on each sublayer's output and a float32 residual stream:
//
//   attention   x -> [q|k|v|gate] GEMM -> convolution + q/k norm + cache append -> attention (window, distance bias, gate)
//               -> output GEMM -> x += norm(.)
//   hgrn2       x -> [q|f|v] GEMM -> recurrence (+ per-head norm) -> output GEMM -> x += norm(.)
//   feed-forward  x -> up GEMM (+ xIELU) -> down GEMM -> x += norm(.)
//
// or, with a norm ahead of each sublayer (pre-norm block), attention alone or beside a Mamba-2 recurrence, then routed experts:
//
//   h -> [q|k|v|head gate or z|x|B|C|dt] GEMM -> q/k norm + rotary positions + cache append -> attention
//                                             -> (convolution +) recurrence -> gated norm
//     -> output GEMM over [heads | recurrence] -> x += ., h = norm(x)
//   h -> router GEMM -> routing -> experts' up GEMM -> experts' down GEMM -> x += ., h = norm(x)
//
// or, with one norm ahead of a mixer and a feed-forward that both read it (parallel block), attention whose values are its
// keys beside routed experts:
//
//   h -> [q|k|shared gate|shared up|router] GEMM -> head split + key append + gated activation + routing
//     -> experts' gated GEMM -> experts' down GEMM;  attention;  output GEMM over [heads | shared expert]
//     -> x += m (.), h = norm(x)
//
// or, with a norm on both sides of each sublayer (sandwich block), attention whose heads' scores are mixed or latent attention,
// then a dense feed-forward, and an average over the depth so far:
//
//   h -> [q|k|v] GEMM -> q/k norm + rotary positions + cache append -> attention with mixed heads
//   h -> [query latent|latent, key part|gate] GEMM -> norms + rotation + latent append -> query GEMM
//        steps:   -> into the latent's space, per head -> attention over the latents -> out of it, per head (+ gate)
//        prompts: latents GEMM to keys and values -> head split -> attention (+ gate)
//     -> output GEMM -> x += norm(.), h = norm(x)
//   h -> up GEMM (+ squared ReLU) -> down GEMM -> x += norm(.), x = depth average, h = norm(x)
//
// Single-token GEMMs leave float32 split-K slabs that the next kernel sums, as in the other families.  The driver around
// this walk (lengths, the captured decode step, sampling, loading) is model.cu's.
#include <string.h>

#include <algorithm>
#include <map>
#include <tuple>

#include "model.h"

using namespace rb;

namespace {

int pad8(int64_t v) { return (int)((v + 7) / 8 * 8); }

// head size of the cache: the next one the tensor-core attention kernels have (bf16), or a multiple of 8 (float32)
int cache_dim(int dtype, int key_dim, int value_dim) {
  const int d = std::max(key_dim, value_dim);
  if (dtype == RB_BF16)
    for (int have : {64, 80, 96, 128, 256})
      if (d <= have) return have;
  return pad8(d);
}

// float32 split-K slabs in m->scratch of x . W^T; returns how many, or 0 when the product has to be a tensor
int slab_count(rb_model* m, int64_t rows, int64_t n, int64_t k) {
  if (m->cfg.dtype != RB_BF16 || rows > 256) return 0;
  const int fit = (int)std::min<size_t>(16, m->scratch_floats / ((size_t)rows * n));
  return std::min(rb_linear_pick_splits(m->ctx, rows, n, k), fit);
}

// stream += norm(x . W^T), and its copy in the model dtype
int sublayer_out(rb_model* m, const void* x, const void* w, int k, const void* gain, int64_t rows) {
  rb_ctx* ctx = m->ctx;
  void* copy = m->cfg.dtype == RB_F32 ? nullptr : m->h;  // float32: the stream itself is the next operand
  const int s = slab_count(m, rows, m->ld, k);
  if (s > 0) {
    RB_TRY(rb_linear_partials(ctx, x, w, m->scratch, rows, m->ld, k, s));
    return rb_add_scaled_norm(ctx, nullptr, m->scratch, s, gain, (float)m->cfg.norm_eps, rows, m->cfg.hidden_size, m->ld, m->stream,
                              copy, m->cfg.dtype);
  }
  RB_TRY(rb_linear(ctx, x, w, nullptr, nullptr, m->sub_out, rows, m->ld, k, RB_ACT_NONE, m->cfg.dtype));
  return rb_add_scaled_norm(ctx, m->sub_out, nullptr, 0, gain, (float)m->cfg.norm_eps, rows, m->cfg.hidden_size, m->ld, m->stream, copy,
                            m->cfg.dtype);
}

int mixer(rb_model* m, const MixLayer& w, int batch, int seq, const int32_t* new_lens) {
  rb_ctx* ctx = m->ctx;
  const int dt = m->cfg.dtype;
  const int64_t rows = (int64_t)batch * seq;
  const float eps = (float)m->cfg.norm_eps;
  const rb_layer_config& c = w.c;
  // input projection: slabs for the consumer to sum at single-token steps, a tensor otherwise
  const int s = seq == 1 ? slab_count(m, rows, w.n_in, m->ld) : 0;
  const void* src = nullptr;
  const float* acc = nullptr;
  if (s > 0) {
    RB_TRY(rb_linear_partials(ctx, m->h, w.in_w, m->scratch, rows, w.n_in, m->ld, s));
    acc = m->scratch;
  } else {
    RB_TRY(rb_linear(ctx, m->h, w.in_w, w.in_b, nullptr, m->mix_in, rows, w.n_in, m->ld, RB_ACT_NONE, dt));
    src = m->mix_in;
  }
  if (c.mixer == RB_MIXER_HGRN2)
    return rb_hgrn2(ctx, src, acc, s, w.n_in, w.f_bias, w.lower, w.out_norm, eps, c.heads, c.key_dim, c.value_dim, batch, seq, m->cache,
                    new_lens, w.state, 0, m->attn, w.mix_k, dt);
  const int kv_heads = c.kv_from < 0 ? c.kv_heads : 0;
  RB_TRY(rb_conv_norm_append(ctx, src, acc, s, w.in_b, w.conv, c.conv_taps, w.q_norm, w.k_norm, eps, batch, seq, c.heads, kv_heads,
                             c.key_dim, c.value_dim, w.n_in, w.kv, w.kv_layer, w.state, new_lens, m->q, s > 0 ? m->gate : nullptr, dt));
  const void* gate = s > 0 ? m->gate : (const char*)m->mix_in + (size_t)w.gate_col * m->es;
  const int64_t gate_ld = s > 0 ? w.n_in - w.gate_col : w.n_in;
  return rb_attention_window(ctx, m->q, w.kv, w.kv_layer, batch, seq, c.heads, c.value_dim, (float)c.scale, c.window, 1, gate, gate_ld,
                             m->attn, w.mix_k, dt);
}

// m->act = act(x . Wup^T): in the GEMM's epilogue, or, when that would leave most SMs idle, from split-K slabs
int mlp_up(rb_model* m, const MixLayer& w, int64_t rows, int act) {
  rb_ctx* ctx = m->ctx;
  const int64_t tiles = (w.mlp_k + 127) / 128;
  if (!ctx->debug_simple && tiles * 4 < (int64_t)ctx->sm_count * 3) {
    const int s = slab_count(m, rows, w.mlp_k, m->ld);
    if (s > 1) {
      RB_TRY(rb_linear_partials(ctx, m->h, w.up, m->scratch, rows, w.mlp_k, m->ld, s));
      return act_from_partials(ctx, m->scratch, s, rows, w.mlp_k, w.mlp_k, false, nullptr, act, m->act, w.act);
    }
  }
  return rb_linear_act(ctx, m->h, w.up, nullptr, m->act, rows, w.mlp_k, m->ld, act, w.act, m->cfg.dtype);
}

// A parallel block on m->h (the stream, normalised): the stream moves on, and m->h is what the next block (gain, or NULL after
// the last) reads.
int parallel_block(rb_model* m, const MixLayer& w, int batch, int seq, const void* next_gain) {
  rb_ctx* ctx = m->ctx;
  const int dt = m->cfg.dtype;
  const int64_t rows = (int64_t)batch * seq;
  const rb_layer_config& c = w.c;
  const bool experts = c.mlp_size > 0;
  // input projection: one set of slabs, router logits included, at single-token steps; otherwise a tensor and float32 logits
  const int s = seq == 1 ? slab_count(m, rows, w.n_in, m->ld) : 0;
  SplitSpec f;
  f.batch = batch; f.s_new = seq; f.q_heads = c.heads; f.kv_heads = c.kv_heads; f.dim = c.key_dim; f.glu_size = c.shared_size;
  f.cache = w.kv; f.layer = w.kv_layer; f.q_out = m->q; f.glu_ld = w.mix_k;
  f.glu_out = c.shared_size > 0 ? (char*)m->attn + (size_t)w.attn_cols * m->es : nullptr;
  RouteSpec r;
  r.experts = c.experts; r.top = c.top; r.groups = c.groups; r.keep = c.keep_groups; r.scale = (float)c.router_scale;
  r.weight = m->route_w; r.list = m->route_list; r.count = m->route_count; r.cap = m->cfg.max_tokens;
  if (s > 0) {
    RB_TRY(rb_linear_partials(ctx, m->h, w.in_w, m->scratch, rows, w.n_in, m->ld, s));
    f.acc = m->scratch; f.n_acc = s; f.bias = w.in_b; f.src_ld = w.n_in;
    r.acc = m->scratch + w.n_main; r.n_acc = s; r.acc_stride = rows * w.n_in; r.z_ld = w.n_in;
  } else {
    RB_TRY(rb_linear(ctx, m->h, w.in_w, w.in_b, nullptr, m->mix_in, rows, w.n_main, m->ld, RB_ACT_NONE, dt));
    f.src = m->mix_in; f.src_ld = w.n_main;
    if (experts) {
      const void* router = (const char*)w.in_w + (size_t)w.n_main * m->ld * m->es;
      const int n = w.n_in - w.n_main;
      if (dt == RB_F32) RB_TRY(rb_linear(ctx, m->h, router, nullptr, nullptr, m->route_z, rows, n, m->ld, RB_ACT_NONE, dt));
      else RB_TRY(rb_linear_partials(ctx, m->h, router, m->route_z, rows, n, m->ld, 1));
      r.acc = m->route_z; r.n_acc = 1; r.z_ld = n;
    }
  }
  RB_TRY(split_and_route(ctx, f, experts ? &r : nullptr, dt));
  if (experts) {
    RB_TRY(rb_moe_gated(ctx, m->h, w.gate, w.up, m->expert_act, rows, c.top, c.experts, r.list, r.count, r.cap, w.ff_p, m->ld, RB_ACT_SILU,
                        m->expert_out, dt));  // (the second product's output is free until then)
    RB_TRY(rb_moe_down(ctx, m->expert_act, w.down, m->expert_out, rows, c.top, c.experts, r.list, r.count, r.cap, m->ld, w.ff_p, dt));
  }
  rb_attention_options o{};
  o.temp_every = c.temp_every; o.temp_coef = (float)c.temp_coef; o.softcap = (float)c.softcap; o.value_dim = c.value_dim;
  o.sink = w.sink; o.out_ld = w.mix_k;
  RB_TRY(rb_attention_general(ctx, m->q, w.kv, w.kv_layer, batch, seq, c.heads, (float)c.scale, &o, m->attn, dt));
  JoinSpec j;
  const int so = slab_count(m, rows, m->ld, w.mix_k);
  if (so > 0) {
    RB_TRY(rb_linear_partials(ctx, m->attn, w.o_w, m->scratch, rows, m->ld, w.mix_k, so));
    j.acc = m->scratch; j.n_acc = so;
  } else {
    RB_TRY(rb_linear(ctx, m->attn, w.o_w, nullptr, nullptr, m->sub_out, rows, m->ld, w.mix_k, RB_ACT_NONE, dt));
    j.y = m->sub_out;
  }
  if (experts) { j.part = m->expert_out; j.weight = m->route_w; j.top = c.top; j.zero = m->route_count; j.n_zero = c.experts; }
  j.mult = (float)c.residual_mult; j.gain = next_gain; j.eps = (float)m->cfg.norm_eps; j.rows = rows; j.width = m->cfg.hidden_size;
  j.ld = m->ld; j.h = m->stream; j.out = next_gain ? m->h : nullptr;
  return add_then_norm(ctx, j, dt);
}

// The mixer of a pre-norm block, from m->h to the operand rows of its output projection (m->attn)
int prenorm_mixer(rb_model* m, const MixLayer& w, int batch, int seq, const int32_t* new_lens) {
  rb_ctx* ctx = m->ctx;
  const int dt = m->cfg.dtype;
  const int64_t rows = (int64_t)batch * seq;
  const float eps = (float)m->cfg.norm_eps;
  const rb_layer_config& c = w.c;
  const int s = seq == 1 ? slab_count(m, rows, w.n_in, m->ld) : 0;
  const void* src = nullptr;
  const float* acc = nullptr;
  if (s > 0) {
    RB_TRY(rb_linear_partials(ctx, m->h, w.in_w, m->scratch, rows, w.n_in, m->ld, s));
    acc = m->scratch;
  } else {
    RB_TRY(rb_linear(ctx, m->h, w.in_w, w.in_b, nullptr, m->mix_in, rows, w.n_in, m->ld, RB_ACT_NONE, dt));
    src = m->mix_in;
  }
  const bool gate_copy = c.head_gate && s > 0;
  RB_TRY(rb_head_norm_rope_append(ctx, src, acc, s, w.in_b, w.n_in, w.q_norm, w.k_norm, eps, w.rope_cos, w.rope_sin, w.rot_dims, batch, seq,
                                  c.heads, c.kv_heads, c.key_dim, c.value_dim, w.kv, w.kv_layer, m->q, gate_copy ? m->gate : nullptr,
                                  gate_copy ? c.heads : 0, dt));
  rb_attention_options o{};
  o.window = c.window; o.chunk = c.chunk; o.value_dim = c.value_dim; o.out_ld = w.mix_k; o.out_scale = (float)c.mixer_scale;
  if (c.head_gate) {
    o.head_gate = 1;
    o.gate = s > 0 ? m->gate : (const char*)m->mix_in + (size_t)w.gate_col * m->es;
    o.gate_ld = s > 0 ? pad8(c.heads) : w.n_in;
  }
  RB_TRY(rb_attention_general(ctx, m->q, w.kv, w.kv_layer, batch, seq, c.heads, (float)c.scale, &o, m->attn, dt));
  if (c.mixer != RB_MIXER_ATTENTION_SSD) return RB_OK;
  const int inner = c.ssd_heads * c.ssd_value_dim;
  RB_TRY(rb_ssd(ctx, src, acc, s, w.n_in, w.x_col, w.conv, w.conv_b, c.conv_taps, w.dt_bias, w.a_log, w.skip, c.ssd_heads, c.ssd_value_dim,
                c.ssd_state, c.ssd_groups, batch, seq, m->cache, new_lens, w.ring, w.state, 0, m->chan, m->rec_out, pad8(inner), dt));
  return rb_gated_group_norm(ctx, m->rec_out, pad8(inner), src, acc, s, w.n_in, w.z_col, w.out_norm, c.ssd_norm_groups, eps,
                             (float)c.ssd_scale, rows, inner, (char*)m->attn + (size_t)w.attn_cols * m->es, w.mix_k, dt);
}

// The experts of a pre-norm block on m->h: their rows, and the routing's weights
int prenorm_experts(rb_model* m, const MixLayer& w, int64_t rows) {
  rb_ctx* ctx = m->ctx;
  const int dt = m->cfg.dtype;
  const rb_layer_config& c = w.c;
  // float32 router logits: slabs when rows are few, otherwise one
  const int s = std::max(1, slab_count(m, rows, w.n_router, m->ld));
  float* z = s > 1 ? m->scratch : m->route_z;
  if (dt == RB_F32) RB_TRY(rb_linear(ctx, m->h, w.router, nullptr, nullptr, z, rows, w.n_router, m->ld, RB_ACT_NONE, dt));
  else RB_TRY(rb_linear_partials(ctx, m->h, w.router, z, rows, w.n_router, m->ld, s));
  rb_route_options o{};
  o.softmax = o.best_of_run = o.renormalise = 1; o.identity = c.identity; o.correction = w.correction; o.identity_weight = m->route_own;
  const int64_t cap = m->cfg.max_tokens;
  RB_TRY(rb_moe_route_general(ctx, z, s, rows * w.n_router, w.n_router, rows, c.experts + c.identity, c.top, c.groups, c.keep_groups, 1.f, &o,
                              m->route_w, m->route_list, m->route_count, cap, dt));
  RB_TRY(rb_moe_up(ctx, m->h, w.up, m->expert_act, rows, c.top, c.experts, m->route_list, m->route_count, cap, w.ff_p, m->ld, RB_ACT_RELU2,
                   m->expert_out, dt));  // (the second product's output is free until then)
  return rb_moe_down(ctx, m->expert_act, w.down, m->expert_out, rows, c.top, c.experts, m->route_list, m->route_count, cap, m->ld, w.ff_p, dt);
}

// A pre-norm block on m->h (the stream, normalised for the mixer); m->h is then what the next block (gain, or NULL after the
// last) reads.
int prenorm_block(rb_model* m, const MixLayer& w, int batch, int seq, const int32_t* new_lens, const void* next_gain) {
  rb_ctx* ctx = m->ctx;
  const int dt = m->cfg.dtype;
  const int64_t rows = (int64_t)batch * seq;
  const rb_layer_config& c = w.c;
  const bool experts = c.mlp_size > 0;
  RB_TRY(prenorm_mixer(m, w, batch, seq, new_lens));
  JoinSpec j;
  j.gain = experts ? w.norm2 : next_gain; j.eps = (float)m->cfg.norm_eps; j.rows = rows; j.width = m->cfg.hidden_size; j.ld = m->ld;
  j.h = m->stream; j.out = j.gain ? m->h : nullptr;
  JoinSpec second = j;
  const int s = slab_count(m, rows, m->ld, w.mix_k);
  if (s > 0) {
    RB_TRY(rb_linear_partials(ctx, m->attn, w.o_w, m->scratch, rows, m->ld, w.mix_k, s));
    j.acc = m->scratch; j.n_acc = s;
  } else {
    RB_TRY(rb_linear(ctx, m->attn, w.o_w, nullptr, nullptr, m->sub_out, rows, m->ld, w.mix_k, RB_ACT_NONE, dt));
    j.y = m->sub_out;
  }
  RB_TRY(add_then_norm(ctx, j, dt));
  if (!experts) return RB_OK;
  RB_TRY(prenorm_experts(m, w, rows));
  second.part = m->expert_out; second.weight = m->route_w; second.top = c.top; second.zero = m->route_count; second.n_zero = c.experts;
  if (c.identity > 0) { second.own = m->route_own; second.own_x = m->h; }
  second.gain = next_gain;
  second.out = next_gain ? m->h : nullptr;
  return add_then_norm(ctx, second, dt);
}

int prenorm_embed(rb_model* m, const uint32_t* tokens, int64_t rows) {
  const rb_model_config& c = m->cfg;
  RB_TRY(rb_embed_norm_stream(m->ctx, m->embed, c.dtype, c.vocab_size, c.hidden_size, m->ld, tokens, rows, m->embed_norm, (float)c.norm_eps,
                              m->stream));
  JoinSpec j;
  j.gain = m->mix[0].norm1; j.eps = (float)c.norm_eps; j.rows = rows; j.width = c.hidden_size; j.ld = m->ld; j.h = m->stream; j.out = m->h;
  j.zero = m->route_count; j.n_zero = kMaxExperts;  // (a call that failed half-way may have left them)
  return add_then_norm(m->ctx, j, c.dtype);
}

// The stream's first value and the first block's input
int parallel_embed(rb_model* m, const uint32_t* tokens, int batch, int seq, const int32_t* new_lens) {
  const rb_model_config& c = m->cfg;
  RB_TRY(rb_embed_positions(m->ctx, m->embed, m->pos, c.max_position_embeddings, c.dtype, c.vocab_size, c.hidden_size, m->ld, tokens,
                            batch, seq, m->cache, new_lens, m->stream));
  JoinSpec j;
  j.gain = m->mix[0].norm1; j.eps = (float)c.norm_eps; j.rows = (int64_t)batch * seq; j.width = c.hidden_size; j.ld = m->ld;
  j.h = m->stream; j.out = m->h;
  j.zero = m->route_count; j.n_zero = kMaxExperts;  // (a call that failed half-way may have left them)
  return add_then_norm(m->ctx, j, c.dtype);
}

// A product of m->h (or another operand): slabs for the consumer to sum at single-token steps, a tensor otherwise
struct Projected {
  const void* src = nullptr;
  const float* acc = nullptr;
  int n_acc = 0;
};
int project(rb_model* m, const void* x, const void* w, const void* bias, void* dst, int64_t rows, int n, int k, int seq, Projected* out) {
  const int s = seq == 1 ? slab_count(m, rows, n, k) : 0;
  if (s > 0) {
    RB_TRY(rb_linear_partials(m->ctx, x, w, m->scratch, rows, n, k, s));
    *out = Projected{nullptr, m->scratch, s};
    return RB_OK;
  }
  RB_TRY(rb_linear(m->ctx, x, w, bias, nullptr, dst, rows, n, k, RB_ACT_NONE, m->cfg.dtype));
  *out = Projected{dst, nullptr, 0};
  return RB_OK;
}

// Attention whose heads' scores are mixed, from m->h to m->attn
int talking_mixer(rb_model* m, MixLayer& w, int batch, int seq) {
  const rb_layer_config& c = w.c;
  if (seq > 1 && w.talk_version != m->params_loaded) {   // the first prompt with these parameters (never a captured step)
    const int n = c.heads * c.heads;
    std::vector<__nv_bfloat16> half(n);
    w.talk_host.resize(n);
    RB_TRY(rb_download(m->ctx, m->cfg.dtype == RB_F32 ? (void*)w.talk_host.data() : (void*)half.data(), w.talk, n * m->es));
    if (m->cfg.dtype == RB_BF16)
      for (int i = 0; i < n; ++i) w.talk_host[i] = __bfloat162float(half[i]);
    w.talk_version = m->params_loaded;
  }
  const int dt = m->cfg.dtype;
  Projected u;
  RB_TRY(project(m, m->h, w.in_w, w.in_b, m->mix_in, (int64_t)batch * seq, w.n_in, m->ld, seq, &u));
  RB_TRY(rb_head_norm_rope_append(m->ctx, u.src, u.acc, u.n_acc, w.in_b, w.n_in, w.q_norm, w.k_norm, (float)m->cfg.norm_eps, w.rope_cos,
                                  w.rope_sin, w.rot_dims, batch, seq, c.heads, c.kv_heads, c.key_dim, c.value_dim, w.kv, w.kv_layer, m->q,
                                  nullptr, 0, dt));
  rb_attention_options o{};
  o.value_dim = c.value_dim; o.out_ld = w.mix_k; o.talk = w.talk; o.sink = w.sink;
  o.talk_host = w.talk_version == m->params_loaded ? w.talk_host.data() : nullptr;
  return rb_attention_general(m->ctx, m->q, w.kv, w.kv_layer, batch, seq, c.heads, (float)c.scale, &o, m->attn, dt);
}

// Latent attention, from m->h to m->attn
int latent_mixer(rb_model* m, const MixLayer& w, int batch, int seq) {
  rb_ctx* ctx = m->ctx;
  const rb_layer_config& c = w.c;
  const int dt = m->cfg.dtype, kv_rank = c.kv_rank;
  const int64_t rows = (int64_t)batch * seq;
  const bool own = c.kv_from < 0;
  // sequences that all start here multiply their latents out; everything else stays in the latent's space
  bool fresh = seq > 1 && w.prompt_kv >= 0;
  for (int b = 0; b < batch && fresh; ++b) fresh = m->cache->host_lens[b] == seq;
  Projected u;
  RB_TRY(project(m, m->h, w.in_w, nullptr, m->mix_in, rows, w.n_in, m->ld, seq, &u));
  const int gates = c.head_gate ? c.heads : c.heads * c.value_dim;
  const bool gate_copy = u.acc != nullptr;
  RB_TRY(rb_latent_append(ctx, u.src, u.acc, u.n_acc, w.n_in, c.q_rank, own ? kv_rank : 0, c.rot_dim, w.dq_norm, w.dkv_norm,
                          (float)m->cfg.norm_eps, w.rope_cos, w.rope_sin, w.rot_dims, c.rot_interleaved, batch, seq, w.kv, w.kv_layer,
                          m->q_latent, own && fresh ? m->latent : nullptr, gate_copy ? m->gate : nullptr, gate_copy ? gates : 0, dt));
  const void* gate = gate_copy ? m->gate : (const char*)m->mix_in + (size_t)w.gate_col * m->es;
  const int64_t gate_ld = gate_copy ? pad8(gates) : w.n_in;
  rb_attention_options o{};
  o.sink = w.sink;
  if (fresh) {
    rb_kv_cache* prompt = m->prompt_kv[w.prompt_kv];
    prompt->pages_per_seq = (seq + kPageTokens - 1) / kPageTokens;
    prompt->max_seq = prompt->pages_per_seq * kPageTokens;
    if (!own) RB_TRY(rb_latent_gather(ctx, w.kv, w.kv_layer, kv_rank, batch, seq, m->latent, dt));
    RB_TRY(rb_linear(ctx, m->q_latent, w.uq, nullptr, nullptr, m->q_raw, rows, w.n_q, w.qr_p, RB_ACT_NONE, dt));
    RB_TRY(rb_linear(ctx, m->latent, w.uk, nullptr, nullptr, m->kv_raw, rows, w.n_kv, w.kr_p, RB_ACT_NONE, dt));
    RB_TRY(rb_latent_heads(ctx, m->q_raw, w.n_q, m->kv_raw, w.n_kv, w.v_col, c.heads, c.key_dim, c.rot_dim, c.value_dim, kv_rank, w.rope_cos,
                           w.rope_sin, w.rot_dims, c.rot_interleaved, batch, seq, w.kv, w.kv_layer, prompt, m->q, dt));
    o.value_dim = c.value_dim; o.out_ld = w.mix_k; o.gate = gate; o.gate_ld = gate_ld; o.head_gate = c.head_gate;
    return rb_attention_general(ctx, m->q, prompt, 0, batch, seq, c.heads, (float)c.scale, &o, m->attn, dt);
  }
  RB_TRY(project(m, m->q_latent, w.uq, nullptr, m->q_raw, rows, w.n_q, w.qr_p, seq, &u));
  RB_TRY(rb_latent_query(ctx, u.src, u.acc, u.n_acc, w.n_q, w.uk, c.heads, c.key_dim, c.rot_dim, kv_rank, w.rope_cos, w.rope_sin, w.rot_dims,
                         c.rot_interleaved, batch, seq, w.kv, m->q, dt));
  o.value_dim = w.kr_p;
  RB_TRY(rb_attention_general(ctx, m->q, w.kv, w.kv_layer, batch, seq, c.heads, (float)c.scale, &o, m->lat_out, dt));
  return rb_latent_output(ctx, m->lat_out, w.uv, c.heads, kv_rank, c.value_dim, gate, gate_ld, c.head_gate, rows, m->attn, w.mix_k, dt);
}

// A sandwich block on m->h (the stream, normalised for the mixer), the l-th; m->h is then what the next block (gain, or NULL after
// the last) reads.  The stream that enters block 0 is the history's first entry.
int sandwich_block(rb_model* m, MixLayer& w, int l, int batch, int seq, const void* next_gain) {
  const rb_model_config& cfg = m->cfg;
  const int64_t rows = (int64_t)batch * seq;
  RB_TRY(w.c.mixer == RB_MIXER_LATENT ? latent_mixer(m, w, batch, seq) : talking_mixer(m, w, batch, seq));
  const bool mlp = w.c.mlp_size > 0;
  SandwichSpec j;
  j.groups = cfg.norm_groups; j.eps = (float)cfg.norm_eps; j.rows = rows; j.width = cfg.hidden_size; j.ld = m->ld;
  j.h_in = l == 0 ? m->history : m->stream; j.h_out = m->stream;
  auto join = [&](const void* x, const void* weight, int k, const void* post, bool last, const void* gain) -> int {
    const int s = slab_count(m, rows, m->ld, k);
    if (s > 0) {
      RB_TRY(rb_linear_partials(m->ctx, x, weight, m->scratch, rows, m->ld, k, s));
      j.acc = m->scratch; j.n_acc = s; j.y = nullptr;
    } else {
      RB_TRY(rb_linear(m->ctx, x, weight, nullptr, nullptr, m->sub_out, rows, m->ld, k, RB_ACT_NONE, cfg.dtype));
      j.y = m->sub_out; j.acc = nullptr; j.n_acc = 0;
    }
    j.post_gain = post;
    if (last) { j.depth = w.depth; j.n_depth = l + 2; j.history = m->history; j.history_stride = (int64_t)cfg.max_tokens * m->ld; }
    j.gain = gain; j.out = gain ? m->h : nullptr;
    return sandwich_join(m->ctx, j, cfg.dtype);
  };
  RB_TRY(join(m->attn, w.o_w, w.mix_k, w.norm1b, !mlp, mlp ? w.norm2 : next_gain));
  if (!mlp) return RB_OK;
  RB_TRY(mlp_up(m, w, rows, RB_ACT_RELU2));
  j.h_in = m->stream;
  return join(m->act, w.down, w.mlp_k, w.norm2b, true, next_gain);
}

int sandwich_embed(rb_model* m, const uint32_t* tokens, int64_t rows) {
  const rb_model_config& c = m->cfg;
  RB_TRY(rb_embed_stream(m->ctx, m->embed, c.dtype, c.vocab_size, c.hidden_size, m->ld, tokens, rows, m->history, nullptr));
  SandwichSpec j;
  j.groups = c.norm_groups; j.eps = (float)c.norm_eps; j.rows = rows; j.width = c.hidden_size; j.ld = m->ld; j.h_in = m->history;
  j.gain = m->mix[0].norm1; j.out = m->h;
  return sandwich_join(m->ctx, j, c.dtype);
}

}  // namespace

int rb::layered_forward(rb_model* m, const uint32_t* tokens, int batch, int seq, const int32_t* new_lens) {
  const rb_model_config& c = m->cfg;
  rb_ctx* ctx = m->ctx;
  const int64_t rows = (int64_t)batch * seq;
  const bool parallel = c.arch == RB_ARCH_VOTAPEL, prenorm = c.arch == RB_ARCH_KUFULIX, sandwich = c.arch == RB_ARCH_FIZADRA;
  if (sandwich) RB_TRY(sandwich_embed(m, tokens, rows));
  else if (parallel) RB_TRY(parallel_embed(m, tokens, batch, seq, new_lens));
  else if (prenorm) RB_TRY(prenorm_embed(m, tokens, rows));
  else
    RB_TRY(rb_embed_stream(ctx, m->embed, c.dtype, c.vocab_size, c.hidden_size, m->ld, tokens, rows, m->stream,
                           c.dtype == RB_F32 ? nullptr : m->h));
  for (size_t l = 0; l < m->mix.size(); ++l) {
    MixLayer& w = m->mix[l];
    const void* next_gain = l + 1 < m->mix.size() ? m->mix[l + 1].norm1 : nullptr;
    if (sandwich) {
      RB_TRY(sandwich_block(m, w, (int)l, batch, seq, next_gain));
    } else if (parallel) {
      RB_TRY(parallel_block(m, w, batch, seq, next_gain));
    } else if (prenorm) {
      RB_TRY(prenorm_block(m, w, batch, seq, new_lens, next_gain));
    } else {
      RB_TRY(mixer(m, w, batch, seq, new_lens));
      RB_TRY(sublayer_out(m, m->attn, w.o_w, w.mix_k, w.norm1, rows));
      if (w.c.mlp_size > 0) {
        RB_TRY(mlp_up(m, w, rows, RB_ACT_XIELU));
        RB_TRY(sublayer_out(m, m->act, w.down, w.mlp_k, w.norm2, rows));
      }
    }
    if (m->layer_trace)
      RB_CUDA(cudaMemcpy2DAsync(m->layer_trace + (size_t)l * rows * c.hidden_size, (size_t)c.hidden_size * 4, m->stream, (size_t)m->ld * 4,
                                (size_t)c.hidden_size * 4, (size_t)rows, cudaMemcpyDeviceToDevice, ctx->stream));
  }
  return RB_OK;
}

int rb::layered_logits(rb_model* m, const int32_t* rows, int seq, int n, float* out) {
  const rb_model_config& c = m->cfg;
  const auto norm = c.arch == RB_ARCH_MALASUN ? rb_scalar_norm_rows : rb_one_plus_norm_rows;
  if (c.arch == RB_ARCH_FIZADRA)
    RB_TRY(rb_group_norm_rows(m->ctx, m->stream, rows, seq, m->norm_w, c.norm_groups, (float)c.norm_eps, n, c.hidden_size, m->ld, m->xn, c.dtype));
  else RB_TRY(norm(m->ctx, m->stream, rows, seq, m->norm_w, (float)c.norm_eps, n, c.hidden_size, m->ld, m->xn, c.dtype));
  if (c.dtype == RB_F32) {
    RB_TRY(rb_linear(m->ctx, m->xn, m->lm_head, nullptr, nullptr, out, n, c.vocab_size, m->ld, RB_ACT_NONE, RB_F32));
  } else {
    for (int r = 0; r < n; r += 256)  // one float32 slab is a float32 product
      RB_TRY(rb_linear_partials(m->ctx, (const char*)m->xn + (size_t)r * m->ld * m->es, m->lm_head, out + (size_t)r * c.vocab_size,
                                std::min(256, n - r), c.vocab_size, m->ld, 1));
  }
  return c.logit_softcap > 0.0 ? rb_soft_cap(m->ctx, out, (int64_t)n * c.vocab_size, (float)c.logit_softcap) : RB_OK;
}

// How many KV splits each attention layer takes: what a captured decode step depends on.
int rb::layered_decode_plan(rb_model* m, int batch) {
  int max_len = 0;
  for (int b = 0; b < batch; ++b) max_len = std::max(max_len, m->cache->host_lens[b]);
  uint32_t plan = 17;
  for (const MixLayer& w : m->mix)
    if (w.kv && w.c.block == RB_BLOCK_SANDWICH)
      plan = plan * 31 + (uint32_t)attention_decode_splits(m->ctx, batch, attention_joint_row_tiles(w.kv, w.c.heads), max_len, 256);
    else if (w.kv)
      plan = plan * 31 + (uint32_t)attention_decode_splits(m->ctx, batch, w.c.kv_heads, attention_walk_len(max_len, w.c.window, w.c.chunk),
                                                           w.kv->head_dim);
  return (int)(plan & 0x7fffffffu);
}

// The layer whose parameters layer l uses (-1: it does not end at one with its own)
static int owner_of(const rb_layer_config* layers, int n, int l) {
  for (int hops = 0; hops <= n; ++hops) {
    if (layers[l].weights_of < 0) return l;
    if (layers[l].weights_of >= n) return -1;
    l = layers[l].weights_of;
  }
  return -1;
}

// What a pre-norm layer may be
static int check_prenorm(const rb_layer_config* layers, int n, int l) {
  const rb_layer_config& y = layers[l];
  const int o = owner_of(layers, n, l);
  RB_REQUIRE(o >= 0, "layer %d: weights_of does not lead to a layer with parameters", l);
  rb_layer_config same = layers[o];
  same.weights_of = y.weights_of;
  RB_REQUIRE(memcmp(&same, &y, sizeof(y)) == 0, "layer %d: differs from layer %d, whose parameters it uses", l, o);
  RB_REQUIRE(y.block == RB_BLOCK_PRE_NORM && (y.mixer == RB_MIXER_ATTENTION || y.mixer == RB_MIXER_ATTENTION_SSD) && y.kv_from < 0 &&
                 (y.mlp_size == 0 || y.mlp_kind == RB_MLP_EXPERTS_RELU2) && y.shared_size == 0,
             "layer %d: block, mixer or feed-forward kind does not belong to this architecture", l);
  RB_REQUIRE(y.heads > 0 && y.kv_heads > 0 && y.heads % y.kv_heads == 0 && y.key_dim > 0 && y.value_dim > 0, "layer %d: bad heads", l);
  if (y.key_dim > 256 || y.value_dim > 256) return fail(RB_ERR_UNIMPLEMENTED, "layer %d: head sizes above 256", l);
  RB_REQUIRE(y.scale > 0.0 && y.window >= 0 && y.window <= (1 << 30) && y.chunk >= 0, "layer %d: bad attention constants", l);
  RB_REQUIRE(y.rot_dims >= 0 && y.rot_dims <= y.key_dim && y.rot_dims % 2 == 0, "layer %d: %d of %d dimensions cannot turn", l, y.rot_dims, y.key_dim);
  RB_REQUIRE(y.mlp_size >= 0, "layer %d: bad feed-forward size", l);
  if (y.mlp_size > 0) {
    const int all = y.experts + y.identity;
    RB_REQUIRE(y.experts > 0 && y.identity >= 0 && y.groups > 0 && all % y.groups == 0 && y.keep_groups > 0 && y.keep_groups <= y.groups &&
                   y.top > 0 && y.top <= all / y.groups * y.keep_groups,
               "layer %d: top %d of %d experts in %d groups of which %d stay", l, y.top, all, y.groups, y.keep_groups);
    if (all > kMaxExperts || y.top > 32) return fail(RB_ERR_UNIMPLEMENTED, "layer %d: more than %d experts or top 32", l, kMaxExperts);
  }
  if (y.mixer != RB_MIXER_ATTENTION_SSD) return RB_OK;
  RB_REQUIRE(y.ssd_heads > 0 && y.ssd_value_dim > 0 && y.ssd_state > 0 && y.ssd_groups > 0 && y.ssd_heads % y.ssd_groups == 0 && y.conv_taps > 0 &&
                 y.ssd_norm_groups > 0 && y.ssd_heads * y.ssd_value_dim % y.ssd_norm_groups == 0,
             "layer %d: bad recurrence sizes", l);
  if (y.ssd_state > 256 || y.ssd_value_dim > 256) return fail(RB_ERR_UNIMPLEMENTED, "layer %d: recurrent states above 256 x 256", l);
  return RB_OK;
}

// What a sandwich layer may be
static int check_sandwich(const rb_layer_config* layers, int l) {
  const rb_layer_config& y = layers[l];
  RB_REQUIRE(y.block == RB_BLOCK_SANDWICH && (y.mixer == RB_MIXER_ATTENTION || y.mixer == RB_MIXER_LATENT) &&
                 (y.mlp_size == 0 || y.mlp_kind == RB_MLP_DENSE_RELU2) && y.mlp_size >= 0,
             "layer %d: block, mixer or feed-forward kind does not belong to this architecture", l);
  RB_REQUIRE(y.heads > 0 && y.key_dim > 0 && y.value_dim > 0 && y.scale > 0.0, "layer %d: bad heads", l);
  RB_REQUIRE(y.rot_dims >= 0 && (y.rot_dims % 2) == 0 && y.rot_dims <= (y.mixer == RB_MIXER_LATENT ? y.rot_dim : y.key_dim),
             "layer %d: %d dimensions cannot turn", l, y.rot_dims);
  if (y.mixer == RB_MIXER_ATTENTION) {
    RB_REQUIRE(y.kv_heads > 0 && y.heads % y.kv_heads == 0 && y.kv_from < 0 && y.talk && y.softmax_one && y.qk_norm && !y.rot_interleaved,
               "layer %d: bad attention", l);
    if (y.key_dim > 256 || y.value_dim > 256) return fail(RB_ERR_UNIMPLEMENTED, "layer %d: head sizes above 256", l);
    return RB_OK;
  }
  RB_REQUIRE(y.q_rank > 0 && y.kv_rank > 0 && y.rot_dim >= 0, "layer %d: bad latent sizes", l);
  if (pad8(y.kv_rank) + y.rot_dim > 960) return fail(RB_ERR_UNIMPLEMENTED, "layer %d: a latent of more than 960 numbers", l);
  if (y.kv_from < 0) return RB_OK;
  RB_REQUIRE(y.kv_from < l && layers[y.kv_from].mixer == RB_MIXER_LATENT && layers[y.kv_from].kv_from < 0,
             "layer %d: kv_from %d is not an earlier layer with a latent of its own", l, y.kv_from);
  const rb_layer_config& o = layers[y.kv_from];
  RB_REQUIRE(o.kv_rank == y.kv_rank && o.rot_dim == y.rot_dim && o.rot_dims == y.rot_dims && o.rot_base == y.rot_base &&
                 o.rot_interleaved == y.rot_interleaved && o.rot_yarn == y.rot_yarn && o.rot_original == y.rot_original &&
                 o.rot_factor == y.rot_factor && o.rot_low == y.rot_low && o.rot_high == y.rot_high,
             "layer %d: its latent or rotation differs from that of layer %d", l, y.kv_from);
  return RB_OK;
}

extern "C" int32_t rb_model_create_layers(rb_ctx* ctx, const rb_model_config* cfg, const rb_layer_config* layers, rb_model** out) {
  RB_REQUIRE(ctx && cfg && layers && out, "rb_model_create_layers: null argument");
  const rb_model_config& c = *cfg;
  const bool parallel = c.arch == RB_ARCH_VOTAPEL, prenorm = c.arch == RB_ARCH_KUFULIX, sandwich = c.arch == RB_ARCH_FIZADRA;
  RB_REQUIRE(c.arch == RB_ARCH_MALASUN || parallel || prenorm || sandwich, "rb_model_create_layers: architecture %d is not described layer by layer", c.arch);
  RB_REQUIRE(c.dtype == RB_BF16 || c.dtype == RB_F32, "rb_model_create_layers: dtype %d unsupported", c.dtype);
  RB_REQUIRE(c.hidden_size > 0 && c.vocab_size > 0 && c.num_hidden_layers > 0, "rb_model_create_layers: bad sizes");
  RB_REQUIRE(c.max_batch > 0 && c.max_seq > 0 && c.max_tokens >= c.max_batch, "rb_model_create_layers: bad capacities");
  // (Malasun: the query / key norm runs over all heads at once, so a head-parallel split would need its sum exchanged per layer)
  if (c.tp_size > 1) return fail(RB_ERR_UNIMPLEMENTED, "rb_model_create_layers: tensor parallelism is not available for this design");
  RB_REQUIRE(!parallel || c.max_position_embeddings > 0, "rb_model_create_layers: learned positions need their number");
  RB_REQUIRE(c.logit_softcap >= 0.0, "rb_model_create_layers: bad logit cap");
  RB_REQUIRE(!sandwich || (c.norm_groups > 0 && c.hidden_size % c.norm_groups == 0), "rb_model_create_layers: %d parts of a row of %d", c.norm_groups,
             c.hidden_size);
  const int L = c.num_hidden_layers;
  for (int l = 0; l < L; ++l) {
    const rb_layer_config& y = layers[l];
    if (prenorm || sandwich) {
      RB_TRY(prenorm ? check_prenorm(layers, L, l) : check_sandwich(layers, l));
      continue;
    }
    RB_REQUIRE(y.block == (parallel ? RB_BLOCK_PARALLEL : RB_BLOCK_POST_NORM) &&
                   (y.mlp_size == 0 || y.mlp_kind == (parallel ? RB_MLP_EXPERTS : RB_MLP_DENSE)),
               "layer %d: block or feed-forward kind does not belong to this architecture", l);
    if (parallel) {
      RB_REQUIRE(y.mixer == RB_MIXER_ATTENTION && y.kv_from < 0 && y.window == 0 && y.key_dim == y.value_dim,
                 "layer %d: a parallel block has attention over every earlier key, whose values are the keys", l);
      RB_REQUIRE(y.temp_every >= 0 && y.softcap >= 0.0 && y.shared_size >= 0, "layer %d: bad constants", l);
      RB_REQUIRE(y.mlp_size > 0 || y.shared_size == 0, "layer %d: a shared expert without experts", l);
      if (y.mlp_size > 0) {
        RB_REQUIRE(y.experts > 0 && y.groups > 0 && y.experts % y.groups == 0 && y.keep_groups > 0 && y.keep_groups <= y.groups &&
                       y.top > 0 && y.top <= y.experts / y.groups * y.keep_groups,
                   "layer %d: top %d of %d experts in %d groups of which %d stay", l, y.top, y.experts, y.groups, y.keep_groups);
        if (y.experts > kMaxExperts || y.top > 32) return fail(RB_ERR_UNIMPLEMENTED, "layer %d: more than %d experts or top 32", l, kMaxExperts);
      }
    }
    RB_REQUIRE(y.mixer == RB_MIXER_ATTENTION || y.mixer == RB_MIXER_HGRN2, "layer %d: unknown mixer %d", l, y.mixer);
    RB_REQUIRE(y.heads > 0 && y.key_dim > 0 && y.value_dim > 0 && y.mlp_size >= 0, "layer %d: bad sizes", l);
    if (y.key_dim > 256 || y.value_dim > 256) return fail(RB_ERR_UNIMPLEMENTED, "layer %d: head sizes above 256", l);
    if (y.mixer != RB_MIXER_ATTENTION) continue;
    RB_REQUIRE(y.kv_heads > 0 && y.heads % y.kv_heads == 0, "layer %d: %d heads over %d key/value heads", l, y.heads, y.kv_heads);
    RB_REQUIRE((parallel || y.conv_taps >= 1) && y.window >= 0 && y.window <= (1 << 30) && y.scale > 0.0, "layer %d: bad attention constants", l);
    if (y.kv_from >= 0) {
      RB_REQUIRE(y.kv_from < l && layers[y.kv_from].mixer == RB_MIXER_ATTENTION && layers[y.kv_from].kv_from < 0,
                 "layer %d: kv_from %d is not an earlier attention layer with keys and values of its own", l, y.kv_from);
      RB_REQUIRE(layers[y.kv_from].kv_heads == y.kv_heads && layers[y.kv_from].key_dim == y.key_dim &&
                     layers[y.kv_from].value_dim == y.value_dim,
                 "layer %d: its key/value heads differ from those of layer %d", l, y.kv_from);
    }
  }

  rb_model* m = new rb_model();
  m->ctx = ctx;
  m->cfg = c;
  m->cfg.tp_size = 1;
  m->cfg.tp_rank = 0;
  if (!parallel) m->cfg.max_position_embeddings = 0x7fffffff;  // positions enter through distances only: no table to outgrow
  m->layered = true;
  m->es = dtype_size(c.dtype);
  m->logits_dtype = RB_F32;
  {
    const char* g = getenv("RAI_B200_GRAPH");  // RAI_B200_GRAPH=0: plain launches for every decode step
    m->use_graph = !(g && g[0] == '0');
  }
  const int W = c.hidden_size, ld = pad8(W), V = c.vocab_size;
  m->ld = ld;
  int st = RB_OK;
  auto A = [&](int64_t elems, void** p) { if (st == RB_OK) st = weight_alloc(m, elems, p); };
  auto at = [&](void* base, int64_t elem_off) { return (void*)((char*)base + elem_off * (int64_t)m->es); };
  auto vec = [&](const std::string& name, int64_t n, void* dst) { add_param(m, name, n, 1, 1, {{0, n, 0, 1, dst, 1}}); };
  auto num = [&](const std::string& name, void* dst) { add_param(m, name, 1, 1, 0, {{0, 1, 0, 1, dst, 1}}); };
  auto mat = [&](const std::string& name, int64_t rows, int64_t cols, void* dst, int64_t dst_ld) {
    add_param(m, name, rows, cols, 2, {{0, rows, 0, cols, dst, dst_ld}});
  };

  A((int64_t)V * ld, &m->embed);
  mat("embed", V, W, m->embed, ld);
  if (parallel) {
    A((int64_t)c.max_position_embeddings * ld, &m->pos);
    mat("pos", c.max_position_embeddings, W, m->pos, ld);
  }
  if (prenorm) {
    A(ld, &m->embed_norm);
    vec("embed.norm", W, m->embed_norm);
  }
  m->mix.resize(L);
  // (key/value heads, cache head size, the values are the keys) -> layers with K and V of their own
  std::map<std::tuple<int, int, bool>, std::vector<int>> geometry;
  auto cached = [&](MixLayer& w, int l, int kv_heads, int head_dim) {
    auto& group = geometry[{kv_heads, head_dim, parallel || w.c.mixer == RB_MIXER_LATENT}];
    w.kv_layer = (int)group.size();
    group.push_back(l);
  };
  int max_in = 8, max_q = 8, max_gate = 8, max_mix = 8, max_mlp = 8, max_experts = 0, max_top = 0, max_ff = 8;
  int max_chan = 0, max_inner = 0, max_gates = 0;
  std::map<std::vector<double>, std::pair<float*, float*>> rotations;  // tables, one set per kind of rotation
  auto turn = [&](MixLayer& w) {
    const rb_layer_config& y = w.c;
    w.rot_dims = y.rot_dims;
    if (y.rot_dims == 0 || st != RB_OK) return;
    const double original = y.rot_original;
    const int positions = (c.max_seq + kPageTokens - 1) / kPageTokens * kPageTokens;   // those of whole pages: padding may sit there
    auto& t = rotations[{(double)y.rot_dims, y.rot_base, original, y.rot_factor, y.rot_low, y.rot_high, (double)y.rot_yarn}];
    if (!t.first) {
      const size_t bytes = (size_t)positions * (y.rot_dims / 2) * sizeof(float);
      st = dev_alloc(m, bytes, (void**)&t.first, false);
      if (st == RB_OK) st = dev_alloc(m, bytes, (void**)&t.second, false);
      if (st == RB_OK)
        st = y.rot_yarn ? rb_rotary_tables_yarn(ctx, y.rot_dims, positions, y.rot_base, y.rot_factor, y.rot_high, y.rot_low, original, t.first, t.second)
                        : rb_rotary_tables(ctx, y.rot_dims, positions, y.rot_base, y.rot_factor, y.rot_low, y.rot_high, original, t.first, t.second);
    }
    w.rope_cos = t.first;
    w.rope_sin = t.second;
  };
  int max_qr = 0, max_kr = 0, max_nq = 0, max_nkv = 0, max_lat = 0, zero_heads = 0;
  std::map<std::pair<int, int>, int> prompt_shapes;   // (heads, head size) -> index into m->prompt_kv
  for (int l = 0; l < L && st == RB_OK; ++l) {
    MixLayer& w = m->mix[l];
    w.c = layers[l];
    const rb_layer_config& y = w.c;
    const std::string pre = "l" + std::to_string(l) + ".", mix = pre + "mix.";
    if (sandwich) {
      const bool latent = y.mixer == RB_MIXER_LATENT, mlp = y.mlp_size > 0;
      auto part = [&](const std::string& name, int64_t n, int64_t row, void* dst) { mat(mix + name, n, W, at(dst, row * ld), ld); };
      turn(w);
      w.mix_k = pad8((int64_t)y.heads * y.value_dim);
      w.mlp_k = pad8(y.mlp_size);
      for (void** p : {&w.norm1, &w.norm1b}) A(ld, p);
      if (mlp) for (void** p : {&w.norm2, &w.norm2b}) A(ld, p);
      A(pad8(l + 2), &w.depth);
      A((int64_t)ld * w.mix_k, &w.o_w);
      if (mlp) { A((int64_t)w.mlp_k * ld, &w.up); A((int64_t)ld * w.mlp_k, &w.down); }
      if (latent) {
        const bool own = y.kv_from < 0;
        const int gates = y.head_gate ? y.heads : y.heads * y.value_dim, nk = y.heads * y.key_dim, nv = y.heads * y.value_dim;
        w.qr_p = pad8(y.q_rank); w.kr_p = pad8(y.kv_rank); w.kv_p = own ? pad8(y.kv_rank + y.rot_dim) : 0;
        w.gate_col = w.qr_p + w.kv_p;
        w.n_in = w.gate_col + pad8(gates);
        w.n_q = pad8((int64_t)y.heads * (y.key_dim + y.rot_dim)); w.v_col = pad8(nk); w.n_kv = w.v_col + pad8(nv);
        A((int64_t)w.n_in * ld, &w.in_w);
        A(w.qr_p, &w.dq_norm);
        if (own) A(w.kr_p, &w.dkv_norm);
        A((int64_t)w.n_q * w.qr_p, &w.uq);
        A((int64_t)w.n_kv * w.kr_p, &w.uk);
        if (y.sink) A(pad8(y.heads), &w.sink);
        if (st != RB_OK) break;
        w.uv = at(w.uk, (int64_t)w.v_col * w.kr_p);
        part("dq", y.q_rank, 0, w.in_w);
        vec(mix + "dq.norm", y.q_rank, w.dq_norm);
        mat(mix + "uq", (int64_t)y.heads * (y.key_dim + y.rot_dim), y.q_rank, w.uq, w.qr_p);
        const int head_dim = c.dtype == RB_BF16 ? (w.kr_p + y.rot_dim + 63) / 64 * 64 : pad8(w.kr_p + y.rot_dim);
        if (own) {
          part("dkv", y.kv_rank + y.rot_dim, w.qr_p, w.in_w);
          vec(mix + "dkv.norm", y.kv_rank, w.dkv_norm);
          cached(w, l, 1, head_dim);
        }
        mat(mix + "uk", nk, y.kv_rank, w.uk, w.kr_p);
        mat(mix + "uv", nv, y.kv_rank, w.uv, w.kr_p);
        if (y.sink) vec(mix + "sink", y.heads, w.sink);
        part("g", gates, w.gate_col, w.in_w);
        const int wide = std::max(y.key_dim + y.rot_dim, y.value_dim), prompt_dim = cache_dim(c.dtype, y.key_dim + y.rot_dim, y.value_dim);
        if (wide <= 256) {
          auto it = prompt_shapes.insert({{y.heads, prompt_dim}, (int)prompt_shapes.size()});
          w.prompt_kv = it.first->second;
          max_q = std::max(max_q, y.heads * prompt_dim);
        }
        max_q = std::max(max_q, y.heads * head_dim);
        max_gate = std::max(max_gate, pad8(gates));
        max_qr = std::max(max_qr, w.qr_p); max_kr = std::max(max_kr, w.kr_p); max_nq = std::max(max_nq, w.n_q);
        max_nkv = std::max(max_nkv, w.n_kv); max_lat = std::max(max_lat, y.heads * w.kr_p);
      } else {
        const int nq = y.heads * y.key_dim, nk = y.kv_heads * y.key_dim, nv = y.kv_heads * y.value_dim, qp = pad8(nq), kp = pad8(nk);
        const int widest = std::max(y.key_dim, y.value_dim), head_dim = c.dtype == RB_BF16 ? (widest + 63) / 64 * 64 : pad8(widest);
        w.n_in = qp + kp + pad8(nv);
        A((int64_t)w.n_in * ld, &w.in_w);
        A(w.n_in, &w.in_b);
        for (void** p : {&w.q_norm, &w.k_norm}) A(pad8(y.key_dim), p);
        A(pad8((int64_t)y.heads * y.heads), &w.talk);
        if (st != RB_OK) break;
        const int n[3] = {nq, nk, nv}, row[3] = {0, qp, qp + kp};
        for (int i = 0; i < 3; ++i) {
          const std::string name(1, "qkv"[i]);
          part(name, n[i], row[i], w.in_w);
          vec(mix + name + ".b", n[i], at(w.in_b, row[i]));
        }
        vec(mix + "q.norm", y.key_dim, w.q_norm);
        vec(mix + "k.norm", y.key_dim, w.k_norm);
        mat(mix + "talk", y.heads, y.heads, w.talk, y.heads);
        cached(w, l, y.kv_heads, head_dim);
        max_q = std::max(max_q, y.heads * head_dim);
        zero_heads = std::max(zero_heads, y.heads);
      }
      if (st != RB_OK) break;
      vec(pre + "norm1", W, w.norm1);
      vec(pre + "norm1b", W, w.norm1b);
      mat(mix + "o", W, (int64_t)y.heads * y.value_dim, w.o_w, w.mix_k);
      if (mlp) {
        vec(pre + "norm2", W, w.norm2);
        vec(pre + "norm2b", W, w.norm2b);
        mat(pre + "mlp.up", y.mlp_size, W, w.up, ld);
        mat(pre + "mlp.down", W, y.mlp_size, w.down, w.mlp_k);
      }
      vec(pre + "dwa", l + 2, w.depth);
      max_in = std::max(max_in, w.n_in);
      max_mix = std::max(max_mix, w.mix_k);
      max_mlp = std::max(max_mlp, w.mlp_k);
      continue;
    }
    if (prenorm) {
      const bool ssd = y.mixer == RB_MIXER_ATTENTION_SSD, own = y.weights_of < 0;
      const int nq = y.heads * y.key_dim, nk = y.kv_heads * y.key_dim, nv = y.kv_heads * y.value_dim, qp = pad8(nq), kp = pad8(nk), vp = pad8(nv);
      const int inner = ssd ? y.ssd_heads * y.ssd_value_dim : 0, bc = ssd ? y.ssd_groups * y.ssd_state : 0, ip = pad8(inner), bp = pad8(bc);
      const int C = ip + 2 * bp, taps = y.conv_taps;
      w.gate_col = qp + kp + vp;
      w.z_col = w.gate_col + (y.head_gate ? pad8(y.heads) : 0);
      w.x_col = w.z_col + ip;
      w.n_in = w.x_col + (ssd ? C + pad8(y.ssd_heads) : 0);
      w.attn_cols = pad8((int64_t)y.heads * y.value_dim);
      w.mix_k = w.attn_cols + ip;
      w.ff_p = pad8(y.mlp_size);
      w.n_router = y.mlp_size > 0 ? pad8(y.experts + y.identity) : 0;
      cached(w, l, y.kv_heads, cache_dim(c.dtype, y.key_dim, y.value_dim));
      if (ssd && st == RB_OK) st = dev_alloc(m, (size_t)c.max_batch * y.ssd_heads * y.ssd_state * y.ssd_value_dim * sizeof(float), (void**)&w.state, true);
      if (ssd && st == RB_OK) st = dev_alloc(m, (size_t)c.max_batch * std::max(1, taps - 1) * C * sizeof(float), (void**)&w.ring, true);
      max_q = std::max(max_q, y.heads * cache_dim(c.dtype, y.key_dim, y.value_dim));
      max_gate = std::max(max_gate, pad8(y.heads));
      max_in = std::max(max_in, w.n_in);
      max_mix = std::max(max_mix, w.mix_k);
      max_chan = std::max(max_chan, C);
      max_gates = std::max(max_gates, y.ssd_heads);
      max_inner = std::max(max_inner, ip);
      if (y.mlp_size > 0) {
        max_experts = std::max(max_experts, w.n_router);
        max_top = std::max(max_top, y.top);
        max_ff = std::max(max_ff, w.ff_p);
      }
      turn(w);
      if (!own) continue;   // parameters: below
      A(ld, &w.norm1);
      A((int64_t)w.n_in * ld, &w.in_w);
      A(w.n_in, &w.in_b);
      A((int64_t)ld * w.mix_k, &w.o_w);
      if (y.qk_norm) {
        A(pad8(y.key_dim), &w.q_norm);
        A(pad8(y.key_dim), &w.k_norm);
      }
      if (ssd) {
        A((int64_t)taps * C, &w.conv);
        A(C, &w.conv_b);
        A(pad8(y.ssd_heads), &w.dt_bias);
        A(pad8(y.ssd_heads), &w.a_log);
        A(pad8(y.ssd_heads), &w.skip);
        A(ip, &w.out_norm);
      }
      if (y.mlp_size > 0) {
        A(ld, &w.norm2);
        A((int64_t)y.experts * w.ff_p * ld, &w.up);
        A((int64_t)y.experts * ld * w.ff_p, &w.down);
        A((int64_t)w.n_router * ld, &w.router);
        A(w.n_router, &w.correction);
      }
      if (st != RB_OK) break;
      vec(pre + "norm1", W, w.norm1);
      const std::string left = ssd ? mix + "left." : mix;
      auto part = [&](const char* name, int n, int col, void* norm) {
        mat(left + name, n, W, at(w.in_w, (int64_t)col * ld), ld);
        vec(left + name + ".b", n, at(w.in_b, col));
        if (norm) vec(left + name + ".norm", y.key_dim, norm);
      };
      part("q", nq, 0, w.q_norm);
      part("k", nk, qp, w.k_norm);
      part("v", nv, qp + kp, nullptr);
      if (y.head_gate) mat(left + "g", y.heads, W, at(w.in_w, (int64_t)w.gate_col * ld), ld);
      mat(left + "o", W, (int64_t)y.heads * y.value_dim, w.o_w, w.mix_k);
      if (ssd) {
        const std::string right = mix + "right.";
        // rows of the file's [z | x | B | C | dt] and where they start here
        const int n[5] = {inner, inner, bc, bc, y.ssd_heads}, to[5] = {w.z_col, w.x_col, w.x_col + ip, w.x_col + ip + bp, w.x_col + C};
        std::vector<Piece> ps, conv, conv_b;
        for (int i = 0, row = 0; i < 5; row += n[i++]) {
          ps.push_back({row, n[i], 0, W, at(w.in_w, (int64_t)to[i] * ld), ld});
          if (i == 0 || i == 4) continue;
          for (int j = 0; j < taps; ++j)  // [channel][tap] in the file, [tap][channel] here
            conv.push_back({row - inner, n[i], j, 1, at(w.conv, (int64_t)j * C + to[i] - w.x_col), 1});
          conv_b.push_back({row - inner, n[i], 0, 1, at(w.conv_b, to[i] - w.x_col), 1});
        }
        add_param(m, right + "in", 2 * inner + 2 * bc + y.ssd_heads, W, 2, ps);
        add_param(m, right + "conv", inner + 2 * bc, taps, 2, conv);
        add_param(m, right + "conv.b", inner + 2 * bc, 1, 1, conv_b);
        vec(right + "dt_bias", y.ssd_heads, w.dt_bias);
        vec(right + "A_log", y.ssd_heads, w.a_log);
        vec(right + "D", y.ssd_heads, w.skip);
        vec(right + "norm", inner, w.out_norm);
        mat(right + "o", W, inner, at(w.o_w, w.attn_cols), w.mix_k);
      }
      if (y.mlp_size > 0) {
        const std::string mlp = pre + "mlp.";
        vec(pre + "norm2", W, w.norm2);
        for (int e = 0; e < y.experts; ++e) {
          const std::string x = mlp + "e" + std::to_string(e) + ".";
          mat(x + "up", y.mlp_size, W, at(w.up, (int64_t)e * w.ff_p * ld), ld);
          mat(x + "down", W, y.mlp_size, at(w.down, (int64_t)e * ld * w.ff_p), w.ff_p);
        }
        mat(mlp + "router", y.experts + y.identity, W, w.router, ld);
        vec(mlp + "correction", y.experts + y.identity, w.correction);
      }
      continue;
    }
    if (parallel) {
      const int nq = y.heads * y.key_dim, nk = y.kv_heads * y.key_dim, qp = pad8(nq), kp = pad8(nk);
      w.glu_p = pad8(y.shared_size);
      w.ff_p = pad8(y.mlp_size);
      w.n_main = qp + kp + 2 * w.glu_p;
      w.n_in = w.n_main + (y.mlp_size > 0 ? pad8(y.experts) : 0);
      w.attn_cols = pad8((int64_t)y.heads * y.value_dim);
      w.mix_k = w.attn_cols + w.glu_p;
      A(ld, &w.norm1);
      A((int64_t)w.n_in * ld, &w.in_w);
      A(w.n_in, &w.in_b);
      A(pad8(y.heads), &w.sink);
      A((int64_t)ld * w.mix_k, &w.o_w);
      if (y.mlp_size > 0) {
        A((int64_t)y.experts * w.ff_p * ld, &w.gate);
        A((int64_t)y.experts * w.ff_p * ld, &w.up);
        A((int64_t)y.experts * ld * w.ff_p, &w.down);
      }
      if (st != RB_OK) break;
      const std::string mlp = pre + "mlp.";
      vec(pre + "norm1", W, w.norm1);
      mat(mix + "q", nq, W, w.in_w, ld);
      vec(mix + "q.b", nq, w.in_b);
      mat(mix + "k", nk, W, at(w.in_w, (int64_t)qp * ld), ld);
      vec(mix + "k.b", nk, at(w.in_b, qp));
      vec(mix + "sink", y.heads, w.sink);
      mat(mix + "o", W, nq, w.o_w, w.mix_k);
      if (y.mlp_size > 0) {
        for (int e = 0; e < y.experts; ++e) {
          const std::string x = mlp + "e" + std::to_string(e) + ".";
          mat(x + "gate", y.mlp_size, W, at(w.gate, (int64_t)e * w.ff_p * ld), ld);
          mat(x + "up", y.mlp_size, W, at(w.up, (int64_t)e * w.ff_p * ld), ld);
          mat(x + "down", W, y.mlp_size, at(w.down, (int64_t)e * ld * w.ff_p), w.ff_p);
        }
        mat(mlp + "router", y.experts, W, at(w.in_w, (int64_t)w.n_main * ld), ld);
      }
      if (y.shared_size > 0) {
        mat(mlp + "shared.gate", y.shared_size, W, at(w.in_w, (int64_t)(qp + kp) * ld), ld);
        mat(mlp + "shared.up", y.shared_size, W, at(w.in_w, (int64_t)(qp + kp + w.glu_p) * ld), ld);
        mat(mlp + "shared.down", W, y.shared_size, at(w.o_w, w.attn_cols), w.mix_k);
      }
      cached(w, l, y.kv_heads, cache_dim(c.dtype, y.key_dim, y.value_dim));
      max_q = std::max(max_q, y.heads * cache_dim(c.dtype, y.key_dim, y.value_dim));
      max_in = std::max(max_in, w.n_in);
      max_mix = std::max(max_mix, w.mix_k);
      if (y.mlp_size > 0) {
        max_experts = std::max(max_experts, pad8(y.experts));
        max_top = std::max(max_top, y.top);
        max_ff = std::max(max_ff, w.ff_p);
      }
      continue;
    }
    A(8, &w.norm1);
    num(pre + "norm1", w.norm1);
    w.mix_k = pad8((int64_t)y.heads * y.value_dim);
    A((int64_t)ld * w.mix_k, &w.o_w);
    if (y.mixer == RB_MIXER_HGRN2) {
      const int hd = y.heads * y.key_dim, p = pad8(hd);
      w.n_in = 2 * p + w.mix_k;
      A((int64_t)w.n_in * ld, &w.in_w);
      A(p, &w.f_bias);
      A(p, &w.lower);
      A(pad8(y.value_dim), &w.out_norm);
      if (st != RB_OK) break;
      mat(mix + "q", hd, W, w.in_w, ld);
      mat(mix + "f", hd, W, at(w.in_w, (int64_t)p * ld), ld);
      vec(mix + "f.b", hd, w.f_bias);
      vec(mix + "lower", hd, w.lower);
      mat(mix + "v", (int64_t)y.heads * y.value_dim, W, at(w.in_w, (int64_t)2 * p * ld), ld);
      vec(mix + "norm", y.value_dim, w.out_norm);
      st = dev_alloc(m, (size_t)c.max_batch * y.heads * y.key_dim * y.value_dim * sizeof(float), (void**)&w.state, true);
    } else {
      const bool own = y.kv_from < 0;
      const int nq = y.heads * y.key_dim, nk = own ? y.kv_heads * y.key_dim : 0, nv = own ? y.kv_heads * y.value_dim : 0;
      const int qp = pad8(nq), kp = pad8(nk), vp = pad8(nv), C = qp + kp + vp, taps = y.conv_taps;
      w.gate_col = C;
      w.n_in = C + w.mix_k;
      A((int64_t)w.n_in * ld, &w.in_w);
      A(w.n_in, &w.in_b);
      A((int64_t)taps * C, &w.conv);
      A(qp, &w.q_norm);
      if (own) A(kp, &w.k_norm);
      if (st != RB_OK) break;
      auto part = [&](const char* name, int n, int col, void* norm) {
        const std::string t = mix + name;
        mat(t, n, W, at(w.in_w, (int64_t)col * ld), ld);
        vec(t + ".b", n, at(w.in_b, col));
        std::vector<Piece> ps;  // [channel][tap] in the file, [tap][channel] here
        for (int j = 0; j < taps; ++j) ps.push_back({0, n, j, 1, at(w.conv, (int64_t)j * C + col), 1});
        add_param(m, t + ".conv", n, taps, 2, ps);
        if (norm) vec(t + ".norm", n, norm);
      };
      part("q", nq, 0, w.q_norm);
      if (own) {
        part("k", nk, qp, w.k_norm);
        part("v", nv, qp + kp, nullptr);
        cached(w, l, y.kv_heads, cache_dim(c.dtype, y.key_dim, y.value_dim));
      }
      mat(mix + "g", (int64_t)y.heads * y.value_dim, W, at(w.in_w, (int64_t)C * ld), ld);
      if (taps > 1) st = dev_alloc(m, (size_t)c.max_batch * (taps - 1) * C * sizeof(float), (void**)&w.state, true);
      max_q = std::max(max_q, y.heads * cache_dim(c.dtype, y.key_dim, y.value_dim));
      max_gate = std::max(max_gate, w.mix_k);
    }
    mat(mix + "o", W, (int64_t)y.heads * y.value_dim, w.o_w, w.mix_k);
    if (y.mlp_size > 0) {
      w.mlp_k = pad8(y.mlp_size);
      A((int64_t)w.mlp_k * ld, &w.up);
      A((int64_t)ld * w.mlp_k, &w.down);
      A(8, &w.act);
      A(8, &w.norm2);
      if (st != RB_OK) break;
      num(pre + "norm2", w.norm2);
      mat(pre + "mlp.up", y.mlp_size, W, w.up, ld);
      mat(pre + "mlp.down", W, y.mlp_size, w.down, w.mlp_k);
      vec(pre + "mlp.act", 2, w.act);
    }
    max_in = std::max(max_in, w.n_in);
    max_mix = std::max(max_mix, w.mix_k);
    max_mlp = std::max(max_mlp, w.mlp_k);
  }
  if (st == RB_OK && prenorm)   // the parameters of another layer; cache, state and ring are the layer's own
    for (int l = 0; l < L; ++l) {
      const int o = owner_of(layers, L, l);
      if (o == l) continue;
      MixLayer& w = m->mix[l];
      const MixLayer own = w;
      w = m->mix[o];
      w.c = own.c; w.kv_layer = own.kv_layer; w.state = own.state; w.ring = own.ring;
    }
  A(parallel || prenorm || sandwich ? ld : 8, &m->norm_w);
  A((int64_t)V * ld, &m->lm_head);
  if (st == RB_OK) {
    if (parallel || prenorm || sandwich) vec("final.norm", W, m->norm_w);
    else num("final.norm", m->norm_w);
    mat("head", V, W, m->lm_head, ld);
    m->vocab_l = V;
  }

  // ---- sequence tables, one cache per attention geometry over them
  if (st == RB_OK) st = kv_cache_create(ctx, nullptr, 0, 1, 8, c.max_batch, c.max_seq, c.dtype, &m->cache);
  for (auto& g : geometry) {
    rb_kv_cache* view = nullptr;
    if (st == RB_OK)
      st = kv_cache_create(ctx, m->cache, (int)g.second.size(), std::get<0>(g.first), std::get<1>(g.first), 0, 0, c.dtype, &view, std::get<2>(g.first));
    if (st != RB_OK) break;
    m->views.push_back(view);
    for (int l : g.second) m->mix[l].kv = view;
  }
  if (st == RB_OK)
    for (MixLayer& w : m->mix)
      if ((w.c.mixer == RB_MIXER_ATTENTION || w.c.mixer == RB_MIXER_LATENT) && w.c.kv_from >= 0) {
        w.kv = m->mix[w.c.kv_from].kv;
        w.kv_layer = m->mix[w.c.kv_from].kv_layer;
      }
  if (st == RB_OK && c.dtype == RB_BF16) {  // split-KV scratch for the worst case: a generation then never allocates
    size_t need = 0;
    for (const MixLayer& w : m->mix)
      if (w.kv) need = std::max(need, (size_t)c.max_batch * w.c.heads * 32 * (w.kv->head_dim + 2) * sizeof(float));
    st = attention_reserve_scratch(ctx, need);
    if (st == RB_OK) st = gemm_reserve_scratch(ctx, (size_t)8 * 64 * std::max(std::max(max_in, max_mlp), ld) * sizeof(float));
  }

  // ---- workspace.  Zeroed: what lies between a row's width and its pitch is multiplied by zero weights and must be finite.
  auto B = [&](size_t bytes, void** p) { if (st == RB_OK) st = dev_alloc(m, bytes, p, true); };
  const size_t MT = c.max_tokens, few = std::min<size_t>(MT, 256);
  B(MT * sizeof(uint32_t), (void**)&m->ids);
  B(MT * ld * sizeof(float), (void**)&m->stream);
  if (c.dtype == RB_F32 && !parallel && !prenorm && !sandwich) m->h = m->stream;
  else B(MT * ld * m->es, &m->h);
  B(MT * max_in * m->es, &m->mix_in);
  B(MT * max_q * m->es, &m->q);
  B(few * max_gate * m->es, &m->gate);
  B(MT * max_mix * m->es, &m->attn);
  B(MT * max_mlp * m->es, &m->act);
  B(MT * ld * m->es, &m->sub_out);
  B((size_t)c.max_batch * ld * m->es, &m->xn);
  B((size_t)c.max_batch * V * sizeof(float), &m->logits);
  B((size_t)c.max_batch * sizeof(uint32_t), (void**)&m->next_ids);
  B(MT * sizeof(int32_t), (void**)&m->last_rows);
  if (parallel || prenorm) B(kMaxExperts * sizeof(int32_t), (void**)&m->route_count);
  if (sandwich) {
    B((size_t)(L + 1) * MT * ld * sizeof(float), (void**)&m->history);
    void* zeros = nullptr;   // sinks of score 0: one more in the softmax denominator
    B((size_t)pad8(zero_heads) * m->es, &zeros);
    for (MixLayer& w : m->mix)
      if (w.c.softmax_one) w.sink = zeros;
  }
  if (max_qr > 0) {
    B(MT * max_qr * m->es, &m->q_latent);
    B(MT * max_kr * m->es, &m->latent);
    B(MT * max_nq * m->es, &m->q_raw);
    // keys and values multiplied out, or each head's weighted latent: never both
    B(MT * std::max(max_nkv, max_lat) * m->es, &m->kv_raw);
    m->lat_out = m->kv_raw;
    const int pages = (int)(MT / kPageTokens) + c.max_batch;   // every sequence of a call may end in a page of its own
    size_t elems = 0;
    for (auto& g : prompt_shapes) elems = std::max(elems, (size_t)pages * kPageTokens * g.first.first * g.first.second);
    void *k = nullptr, *v = nullptr, *table = nullptr;
    if (!prompt_shapes.empty()) { B(elems * m->es, &k); B(elems * m->es, &v); }
    B((size_t)pages * sizeof(int32_t), &table);
    std::vector<int32_t> in_order(pages);
    for (int i = 0; i < pages; ++i) in_order[i] = i;
    if (st == RB_OK) st = rb_upload(ctx, table, in_order.data(), in_order.size() * sizeof(int32_t));
    if (st == RB_OK) RB_CUDA(cudaStreamSynchronize(ctx->stream));   // (the vector dies with this frame)
    m->prompt_kv.resize(prompt_shapes.size(), nullptr);
    for (auto& g : prompt_shapes) {
      if (st != RB_OK) break;
      rb_kv_cache* p = new rb_kv_cache(m->cache);
      p->ctx = ctx; p->layers = 1; p->kv_heads = g.first.first; p->head_dim = g.first.second; p->dtype = c.dtype; p->max_batch = c.max_batch;
      p->num_pages = pages; p->k = k; p->v = v; p->block_table = (int32_t*)table; p->seq_lens = m->cache->seq_lens; p->slots = m->cache->slots;
      m->prompt_kv[g.second] = p;
    }
  }
  if (max_inner > 0) {
    B(MT * max_chan * m->es + (size_t)c.max_batch * max_gates * 2 * sizeof(float), &m->chan);
    B(MT * max_inner * m->es, &m->rec_out);
  }
  if (max_experts > 0) {
    B(MT * max_experts * sizeof(float), (void**)&m->route_z);
    B(MT * max_top * sizeof(float), (void**)&m->route_w);
    B(MT * sizeof(float), (void**)&m->route_own);
    B(MT * max_experts * sizeof(int32_t), (void**)&m->route_list);
    B(MT * max_top * max_ff * m->es, &m->expert_act);
    B(MT * max_top * ld * m->es, &m->expert_out);
  }
  B((size_t)c.max_batch * sizeof(int32_t), (void**)&m->new_lens);
  if (c.dtype == RB_BF16) {
    m->scratch_floats = (size_t)16 * few * std::max({max_in, max_mlp, ld, max_experts, max_nq});
    B(m->scratch_floats * sizeof(float), (void**)&m->scratch);
  }
  if (st != RB_OK) { rb_model_destroy(m); return st; }
  RB_CUDA(cudaStreamSynchronize(ctx->stream));
  *out = m;
  return RB_OK;
}
