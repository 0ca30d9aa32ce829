// The decoder behind the opaque rb_model handle: parameters, caches, workspace and the captured decode step.  Shared by
// the two layer walks: the four transformer families (model.cu) and the designs described layer by layer (layered.cu).
#pragma once
#include <map>
#include <string>
#include <vector>

#include "ctx.h"

namespace rb {

// One rectangular piece of a reference parameter and where it lands in this rank's buffers.
struct Piece {
  int64_t src_row0, rows, src_col0, cols;
  void* dst;
  int64_t dst_ld;  // elements
};
struct ParamSpec {
  int64_t rows, cols;  // full shape of the reference parameter (cols = 1 for vectors)
  int rank;            // 1 or 2
  std::vector<Piece> pieces;
  bool loaded = false;
};

struct LayerW {
  void *qkv = nullptr, *qkv_b = nullptr;
  void *o = nullptr, *o_b = nullptr;
  void *gate = nullptr, *up = nullptr, *fc1_b = nullptr;  // phi2: gate = fc1
  void *down = nullptr, *down_b = nullptr;                // phi2: down = fc2
  void *ln1_w = nullptr, *ln1_b = nullptr, *ln2_w = nullptr;
};

struct Pending {  // terms still to be added to the residual stream
  const float* acc = nullptr;
  int n_acc = 0;
  const void* acc_bias = nullptr;
  const void* add = nullptr;
  bool exchange = false;  // the term is one rank's share: the norm point sums it over the tensor-parallel group
  bool any() const { return (acc && n_acc > 0) || add || exchange; }
};

// One layer of a design that is described layer by layer.
struct MixLayer {
  rb_layer_config c{};
  int n_in = 0;                // columns of the fused input projection (every part padded to a multiple of 8)
  int gate_col = 0;            // attention: where the output gate's columns start
  int mix_k = 0, mlp_k = 0;    // padded K of the output projection and of the down projection
  void *in_w = nullptr, *in_b = nullptr, *o_w = nullptr, *norm1 = nullptr, *norm2 = nullptr;
  void *conv = nullptr, *q_norm = nullptr, *k_norm = nullptr;         // attention
  void *f_bias = nullptr, *lower = nullptr, *out_norm = nullptr;      // hgrn2
  void *up = nullptr, *down = nullptr, *act = nullptr;
  // parallel block (one fused input projection [q | k | shared gate | shared up | router], one fused output projection over
  // [heads | shared expert's inner row]) with experts stacked in gate, up and down
  int n_main = 0, attn_cols = 0, glu_p = 0, ff_p = 0;  // columns before the router's; of the heads; padded inner sizes
  void *sink = nullptr, *gate = nullptr;
  // pre-norm block (fused input projection [q | k | v | head gate] or [q | k | v | z | x | B | C | dt], fused output projection
  // over [heads | recurrence], both with the parts that the layer has)
  int z_col = 0, x_col = 0, n_router = 0, rot_dims = 0;
  const float *rope_cos = nullptr, *rope_sin = nullptr;
  void *conv_b = nullptr, *dt_bias = nullptr, *a_log = nullptr, *skip = nullptr, *router = nullptr, *correction = nullptr;
  float* ring = nullptr;       // Mamba-2: earlier channel values [slot][taps - 1][channels]
  // sandwich block: norms behind the sublayers, weights of the depth average; head-mixing attention (zero: sinks of score 0);
  // latent attention (fused input projection [query latent | latent, key part | gate])
  void *norm1b = nullptr, *norm2b = nullptr, *depth = nullptr, *talk = nullptr;
  void *dq_norm = nullptr, *dkv_norm = nullptr, *uq = nullptr, *uk = nullptr, *uv = nullptr;   // uk, uv: one matrix [keys | values]
  std::vector<float> talk_host;   // as of talk_version of rb_model::params_loaded
  int64_t talk_version = -1;
  int qr_p = 0, kv_p = 0, kr_p = 0, n_q = 0, n_kv = 0, v_col = 0;   // padded sizes: latents, their columns, heads multiplied out
  int prompt_kv = -1;          // index into rb_model::prompt_kv; -1: prompts, too, attend in the latent's space
  rb_kv_cache* kv = nullptr;   // the cache (of this layer's geometry) its keys and values are in, and the layer there
  int kv_layer = 0;
  float* state = nullptr;      // attention: ring of projected values [slot][taps - 1][channels]; recurrences: [slot][head][key][value]
};

}  // namespace rb

struct rb_model {
  rb_ctx* ctx = nullptr;
  rb_model_config cfg{};
  int d = 0, nq_l = 0, nkv_l = 0, nqkv_l = 0, inter_l = 0, vocab_l = 0;
  std::vector<int> q_head_src;  // global q head of local head j, or -1 for padding
  int kv_head0 = 0;             // first global kv head of this rank
  size_t es = 2;
  std::vector<rb::LayerW> layers;
  void *embed = nullptr, *norm_w = nullptr, *norm_b = nullptr, *lm_head = nullptr, *lm_head_b = nullptr;
  float *rope_cos = nullptr, *rope_sin = nullptr;
  rb_kv_cache* cache = nullptr;
  std::vector<void*> owned;
  std::vector<std::string> names;
  std::map<std::string, rb::ParamSpec> params;
  int64_t param_bytes = 0;
  int64_t params_loaded = 0;   // grows with every parameter that is loaded
  // workspace
  uint32_t* ids = nullptr;
  void *h = nullptr, *xn = nullptr, *tmp = nullptr, *qkv = nullptr, *q = nullptr, *attn = nullptr, *act = nullptr;
  void *last_h = nullptr, *logits = nullptr, *logits_g = nullptr;
  uint32_t* next_ids = nullptr;
  int32_t* last_rows = nullptr;           // the rows of a call whose logits are wanted [max_tokens]
  std::vector<int32_t> last_rows_host;    // outlives the asynchronous upload
  float* scratch = nullptr;  // split-K partials
  size_t scratch_floats = 0;
  void* comm = nullptr;
  // peer-memory exchange for decode-sized allreduces (see TpPeers); xchg_base is this rank's region
  TpPeers peers{};
  void* xchg_base = nullptr;
  int xchg_index = 0;  // exchanges launched so far in this forward pass (an even number per pass: two per layer)
  void* peer_base[kTpMaxRanks] = {};
  bool use_exchange = false;
  // RAI_B200_TP_FUSED_GATE=1: a sharded gate/up GEMM sums its split-K slabs and applies activation and gating in its
  // own epilogue.  Off by default: measured slower than split-K partials plus the small finishing kernel, whose many
  // blocks read the slabs with far more parallelism.
  bool fused_gate = false;
  // Developer builds only (-DRB_DEBUG_AIDS, a library file of its own): RAI_B200_SHARD_ONLY=1 runs one rank's shard
  // without its peers to time the per-rank kernels; its outputs are not the model's.  Always false otherwise.
  bool shard_only = false;
  // One decode step (advance lengths, forward of the tokens in `ids`, argmax back into `ids`)
  // captured as a CUDA graph and replayed; re-captured when the batch or the launch plan changes.
  cudaGraphExec_t step_graph = nullptr;
  int graph_batch = 0, graph_plan = 0;
  int eager_warm_batch = 0, eager_warm_plan = 0;
  int64_t graph_launches = 0;
  bool use_graph = true;
  cudaEvent_t ev_in = nullptr, ev_out = nullptr;
  // sampling of the generation entry points (rb_model_set_sampling): repeat penalty over a ring of the
  // last `rep_last_n` tokens fed per sequence, and the end-of-sequence rule
  float rep_penalty = 0.f;
  int rep_last_n = 0;
  int32_t eos = -1;
  int32_t *hist = nullptr, *hist_count = nullptr;
  uint8_t* finished = nullptr;
  // designs described layer by layer (layered.cu): `cache` then holds only the sequence tables
  bool layered = false;
  std::vector<rb::MixLayer> mix;
  std::vector<rb_kv_cache*> views;        // one cache per attention geometry
  int ld = 0;                             // pitch of the residual stream (hidden_size padded to a multiple of 8)
  float* stream = nullptr;                // float32 residual stream [max_tokens][ld]
  void *mix_in = nullptr, *gate = nullptr, *sub_out = nullptr;
  void *pos = nullptr;                    // learned position vectors
  void *embed_norm = nullptr;             // weight of the norm on the embedding
  // routing of a call's rows to experts: logits, weights of the choices, each expert's list of them, and their rows
  float *route_z = nullptr, *route_w = nullptr;
  int32_t *route_list = nullptr, *route_count = nullptr;
  void *expert_act = nullptr, *expert_out = nullptr;
  float* route_own = nullptr;             // weight of a row's identity experts
  void *chan = nullptr, *rec_out = nullptr;  // a recurrence's channels after their convolution, and its output
  // sandwich blocks: the embedding and every layer's result [layers + 1][max_tokens][ld]; latent attention's intermediate rows,
  // and where a prompt's keys and values go when its latents are multiplied out (pages in order, one buffer for all layers)
  float* history = nullptr;
  void *q_latent = nullptr, *latent = nullptr, *q_raw = nullptr, *kv_raw = nullptr, *lat_out = nullptr;
  std::vector<rb_kv_cache*> prompt_kv;
  float* layer_trace = nullptr;
  int logits_dtype = RB_BF16;
  int32_t* new_lens = nullptr;            // device [max_batch]: tokens each sequence feeds in this call
  std::vector<int32_t> new_lens_host;     // outlives the asynchronous upload
};

namespace rb {
int dev_alloc(rb_model* m, size_t bytes, void** out, bool zero);
int weight_alloc(rb_model* m, int64_t elems, void** out);
void add_param(rb_model* m, const std::string& name, int64_t rows, int64_t cols, int rank, std::vector<Piece> pieces);
// The launches between the token ids and the final residual stream of a layered design, and the logits of `n` of its rows
// (row indices on the device, or NULL: the last row of each of the `n` sequences of `seq` rows).
int layered_forward(rb_model* m, const uint32_t* tokens, int batch, int seq, const int32_t* new_lens);
int layered_logits(rb_model* m, const int32_t* rows, int seq, int n, float* out);
int layered_decode_plan(rb_model* m, int batch);
}  // namespace rb
