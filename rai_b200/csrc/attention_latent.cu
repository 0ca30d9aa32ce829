// Latent attention on the kernel of attention_joint.cuh, and the choice between that kernel's shapes and the plain kernels.
#include "attention_joint.cuh"

namespace rb {

using joint::Shape;

int attention_talk_tc(rb_ctx* ctx, const joint::Params& p, rb_kv_cache* c, int layer, int batch, int max_len);

namespace {

int attention_latent_tc(rb_ctx* ctx, const joint::Params& p, rb_kv_cache* c, int layer, int batch, int max_len) {
  const int rows = p.s_new * p.group;
  // 64 keys per tile, all warps on one head; 16-dimension tiles per warp, 8-row tiles
#define RB_LATENT(DW, NT) return joint::launch<Shape<64, 8, 1, DW, NT, true>>(ctx, c, p, layer, batch, max_len)
#define RB_ROWS(DW) \
  if (rows <= 8) RB_LATENT(DW, 1); \
  if (rows <= 16) RB_LATENT(DW, 2); \
  if (rows <= 32 || p.nbk > 8) RB_LATENT(DW, 4); \
  RB_LATENT(DW, 8)
  if (p.value_dim <= 128) { RB_ROWS(1); }
  if (p.value_dim <= 256) { RB_ROWS(2); }
  if (p.value_dim <= 512) { RB_ROWS(4); }
#undef RB_ROWS
#undef RB_LATENT
  return RB_ERR_UNIMPLEMENTED;
}

}  // namespace

int attention_joint_row_tiles(const rb_kv_cache* c, int q_heads) {
  if (!c->shared()) return 1;
  const int rows = c->head_dim > 512 ? 32 : 64;
  return (q_heads + rows - 1) / rows;
}

bool attention_joint_takes(const rb_kv_cache* c, const AttnExtra& x) {
  if (c->dtype != RB_BF16 || (c->head_dim % 64) != 0 || x.alibi || x.gate || x.temp_every || x.softcap != 0.f || x.out_scale != 1.f) return false;
  return x.talk ? !c->shared() : c->shared() && c->kv_heads == 1 && x.value_dim <= 512;
}

int attention_joint(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads, float scale, void* out,
                    const AttnExtra& x) {
  if (x.talk && ctx->attn_tc && attention_mix_tc_takes(c, s_new, q_heads, q, x))
    return attention_mix_tc(ctx, q, c, layer, batch, s_new, q_heads, scale, out, x);
  joint::Params p{};
  p.q = (const bf16*)q; p.block_table = c->block_table; p.seq_lens = c->seq_lens; p.pages_per_seq = c->pages_per_seq; p.s_new = s_new;
  p.D = c->head_dim; p.q_heads = q_heads; p.kv_heads = c->kv_heads; p.group = q_heads / c->kv_heads;
  p.nbk = c->head_dim / 64; p.nbv = (x.value_dim + 63) / 64;
  p.window = x.window > 0 ? x.window : 1 << 30; p.chunk = x.chunk; p.value_dim = x.value_dim; p.scale_log2 = scale * joint::kLog2e;
  p.talk = (const bf16*)x.talk; p.sink = (const bf16*)x.sink; p.out = (bf16*)out; p.out_ld = x.out_ld;
  p.split_count = c->split_count; p.status = ctx->status_dev; p.wait_cycles = ctx->local_wait_cycles();
  int max_len = 0;
  for (int b = 0; b < batch; ++b) max_len = std::max(max_len, c->host_lens[b]);
  max_len = attention_walk_len(max_len, x.window, x.chunk);
  const int st = x.talk ? attention_talk_tc(ctx, p, c, layer, batch, max_len) : attention_latent_tc(ctx, p, c, layer, batch, max_len);
  if (st != RB_ERR_UNIMPLEMENTED) return st;
  return x.talk ? attention_talk_simple(ctx, q, c, layer, batch, s_new, q_heads, scale, out, c->dtype, x)
                : attention_simple(ctx, q, c, layer, batch, s_new, q_heads, scale, out, c->dtype, &x);
}

}  // namespace rb
