// Attention whose heads' scores are mixed before the softmax, on the kernel of attention_joint.cuh: which of its shapes fits.
#include "attention_joint.cuh"

namespace rb {

using joint::Shape;

int attention_talk_tc(rb_ctx* ctx, const joint::Params& p, rb_kv_cache* c, int layer, int batch, int max_len) {
  const bool wide = p.value_dim > 128;
  const int G = p.kv_heads, rows = p.s_new * p.group;   // rows per key/value head
  // 32 keys per tile, single tokens 64; warps per key/value head, heads per team, 16-dimension tiles per warp, 8-row tiles
#define RB_TALK(WG, GP, DW, MANY) \
  return rows <= 8 ? joint::launch<Shape<64, WG, GP, DW, 1, false>>(ctx, c, p, layer, batch, max_len) \
                   : joint::launch<Shape<32, WG, GP, DW, MANY, false>>(ctx, c, p, layer, batch, max_len)
  if (G == 1) { if (wide) RB_TALK(8, 1, 2, 8); RB_TALK(8, 1, 1, 8); }
  if (G == 2) { if (wide) RB_TALK(4, 1, 4, 8); RB_TALK(4, 1, 2, 8); }
  if (G <= 4) { if (wide) RB_TALK(2, 1, 8, 4); RB_TALK(2, 1, 4, 8); }
  if (G <= 8) { if (wide) RB_TALK(1, 1, 16, 2); RB_TALK(1, 1, 8, 4); }
  if (G <= 16 && !wide)
    return rows <= 8 ? joint::launch<Shape<32, 1, 2, 8, 1, false>>(ctx, c, p, layer, batch, max_len)
                     : joint::launch<Shape<32, 1, 2, 8, 2, false>>(ctx, c, p, layer, batch, max_len);
#undef RB_TALK
  if (G <= 16) return joint::launch<Shape<32, 1, 2, 16, 1, false>>(ctx, c, p, layer, batch, max_len);
  if (G <= 32 && !wide) return joint::launch<Shape<32, 1, 4, 8, 1, false>>(ctx, c, p, layer, batch, max_len);
  return RB_ERR_UNIMPLEMENTED;
}

}  // namespace rb
