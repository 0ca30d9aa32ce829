// Internal definition of the context and the KV cache behind the opaque handles of the C ABI.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>

#include <map>
#include <tuple>
#include <vector>

#include "common.cuh"

struct rb_ctx {
  int device = 0;
  cudaStream_t own_stream = nullptr;
  cudaStream_t stream = nullptr;
  int sm_count = 148;
  uint32_t* status_dev = nullptr;  // 4 words, see rb_status_word
  int64_t launches = 0;
  // Tensor maps are keyed by (base pointer, rows, cols, row stride in elements, box rows).
  std::map<std::tuple<const void*, int64_t, int64_t, int64_t, int>, CUtensorMap> tmaps;
  bool pdl = true;            // RAI_B200_PDL=0 turns programmatic dependent launch off (debugging aid)
  // shared memory a decode-sized GEMM spends on its operand ring (RAI_B200_GEMM_RING_KB overrides)
  size_t gemm_ring_bytes = 200 * 1024;
  bool attn_tc = true;        // RAI_B200_ATTN_TC=0: prefill attention on the mma.sync kernel for every head size (debugging aid)
  bool gemm_reduce = true;    // RAI_B200_GEMM_REDUCE=0: rb_linear / rb_gated_linear never split K inside the kernel (debugging aid)
  float* gemm_scratch = nullptr;   // float32 slabs of the GEMMs that reduce split-K inside the kernel; grow-only
  size_t gemm_scratch_bytes = 0;
  uint32_t* gemm_tile_count = nullptr;  // [2][kGemmMaxReduceTiles] arrival / done counters of those GEMMs, self-resetting
  long long wait_budget_cycles = 2000000000LL;  // give-up time of a device-side wait for ANOTHER GPU (rb_set_wait_budget_us)
  // Waits inside one kernel (operand rings, accumulators, sibling blocks) may begin before the kernel's predecessor
  // has finished, and that predecessor may itself be waiting for a peer: they get four times the budget, so that
  // when a peer never arrives it is the exchange that reports it, not a bystander further down the stream.
  long long local_wait_cycles() const { return wait_budget_cycles > (1LL << 60) ? wait_budget_cycles : 4 * wait_budget_cycles; }
  int tmap_cache_limit = 4096;  // tensor maps kept before the cache is emptied
  // argmax across blocks: running best (key << 32 | index) and arrival count per row; self-resetting
  unsigned long long* argmax_best = nullptr;
  unsigned int* argmax_count = nullptr;
  float* chunk_scratch = nullptr;   // states between the pieces of a recurrence that is run piecewise; grow-only
  size_t chunk_scratch_bytes = 0;
  // split-KV partials of the decode attention: grown on demand, owned by the context (one stream at a time)
  bool pool_ready = false;  // the device's default memory pool has been told to keep freed blocks
  float* attn_scratch = nullptr;
  size_t attn_scratch_bytes = 0;
  std::vector<void*> retired;  // outgrown scratch buffers, kept until rb_destroy (captured graphs may still name them)
  std::vector<struct rb_kv_cache*> caches;  // live caches, for the clean-up after a device-side give-up
  double cycles_per_us = 1965.0;  // SM clock, to turn a wait budget in microseconds into cycles
  bool debug_simple = false;
  bool debug_no_fuse = false;  // RAI_B200_FUSE_ROPE=0
  bool debug_simple_gemm = false, debug_simple_attn = false;  // RAI_B200_SIMPLE_GEMM / _ATTN: one kernel family only  // RAI_B200_SIMPLE=1: route bf16 through the plain kernels (debugging aid)
  // Optional per-launch timing (rb_profile_start / rb_profile_read): an event pair around each launch.
  struct ProfRec { int cls; cudaEvent_t a, b; double bytes, flops; };
  bool profiling = false;
  std::vector<ProfRec> prof;
};

// Pages of 64 tokens.  K and V each: [layer][page][kv_head][64][head_dim] in the cache dtype.
//
// A design whose layers differ in head counts or sizes has one cache per geometry over ONE set of sequences: the
// first owns the tables (block table, lengths, state slots), the others are views that share them (`tables`).  A
// cache with layers == 0 is only the tables.
constexpr int kLatentRowTiles = 16;   // arrival counters per sequence of a cache with one head that is key and value

struct rb_kv_cache {
  explicit rb_kv_cache(rb_kv_cache* shared = nullptr)
      : tables(shared), host_lens(shared ? shared->host_lens : own_lens) {}
  rb_kv_cache* tables = nullptr;   // the cache whose tables this one uses; null = its own
  std::vector<int32_t> own_lens;
  rb_ctx* ctx = nullptr;
  int layers = 0, kv_heads = 0, head_dim = 0, max_batch = 0, max_seq = 0, dtype = RB_BF16;
  int pages_per_seq = 0, num_pages = 0;
  int window = 1 << 30;  // sliding-window width of the attention mask (rb_kv_cache_set_window); 2^30 = none
  void* k = nullptr;
  void* v = nullptr;               // == k: the values are the keys
  bool shared() const { return k == v; }
  int32_t* block_table = nullptr;  // device [max_batch][pages_per_seq]
  int32_t* seq_lens = nullptr;     // device [max_batch]
  int32_t* slots = nullptr;        // device [max_batch]: where sequence b keeps its recurrent and convolution state
  std::vector<int32_t> host_table, host_slots;  // host copies of block_table and slots
  uint32_t* split_count = nullptr;  // device [max_batch][kv_heads] (one shared head: [max_batch][kLatentRowTiles]): arrivals of a split decode attention; self-resetting
  std::vector<int32_t>& host_lens;
  size_t split_counters() const { return (size_t)max_batch * (shared() && kv_heads == 1 ? kLatentRowTiles : kv_heads); }
  size_t layer_stride_elems() const { return (size_t)num_pages * kv_heads * 64 * head_dim; }
};

// Peer-memory exchange of a tensor-parallel group for decode-sized allreduces (exchange_norm_kernel, one block per
// row).  Flag-array form: every rank stores its partial row into its own place in every PEER's exchange buffer (posted
// stores over NVLink), raises the flag of (source rank, row) in every peer's flag array with a system-scope release,
// waits (bounded) for that row's flag from every peer - not for the other rows - and sums the copies in its own memory
// and its own row in rank order, the same on every rank.  The two flag-in-data forms need no flag array: every
// 8-byte word carries 4 bytes of payload and the exchange number (see the kernel).  Two slots, chosen by the parity
// of an exchange number kept on the device, so replayed CUDA graphs need no new arguments: launches alternate
// between two local counters (a launch reads one and sets the other for its successor), so no kernel changes a word
// its own blocks are still reading.  Slot n & 1 is free again when exchange n + 2 starts: a rank gets there only
// after every rank has delivered its rows of exchange n + 1, which a rank does only after its own exchange n has
// completed.
constexpr int kGemmMaxReduceTiles = 256;

constexpr int kTpMaxRanks = 8;
constexpr int kTpMaxRows = 256;
// Forms of the exchange (see exchange_norm_kernel): how arrival is signalled and which way the rows travel.
enum TpForm : int { kTpFlagArray = 0, kTpInDataDirect = 1, kTpInDataTwoHop = 2 };
constexpr int kTpDirectRanks = 2;      // widest group that sends flag-in-data words straight to every peer
constexpr int kTpTwoHopRanks = 8;      // widest group that takes the two-hop form of them by default
constexpr size_t kTpFlagBytes = (size_t)2 * kTpMaxRanks * kTpMaxRows * sizeof(uint32_t);  // [2 slots][source rank][row]
struct TpPeers {
  const void* xbuf[kTpMaxRanks];   // every rank's exchange buffer (own included), [2 slots][size sources][kTpMaxRows][hidden]
                                   // (flag-in-data form: the same shape in 8-byte words of 2 elements + the exchange number)
  uint32_t* flags[kTpMaxRanks];    // every rank's flag array, [2][kTpMaxRanks][kTpMaxRows]
  uint32_t* seq;                   // local: two exchange counters 128 bytes apart, seq[0] for even launches, seq[32] for odd
  int rank, size;
  int form;                        // a TpForm
  int64_t slot_elems;              // kTpMaxRows * hidden
};

namespace rb {
// api.cu: layers >= 0; `shared` makes a view over another cache's sequences (max_batch and max_seq are then its)
// (values_are_keys: one set of pages for both)
int kv_cache_create(rb_ctx* ctx, rb_kv_cache* shared, int layers, int kv_heads, int head_dim, int max_batch, int max_seq, int dtype,
                    rb_kv_cache** out, bool values_are_keys = false);
// sequences order[0 .. max_batch) (a permutation) become 0, 1, ...: pages, slots and lengths move with them
int kv_cache_permute(rb_kv_cache* c, const std::vector<int32_t>& order);
constexpr int kPageTokens = 64;
constexpr int kArgmaxRows = 4096;  // rows one argmax launch can reduce across blocks

// Brackets one kernel launch with CUDA events when profiling is on; `bytes` / `flops` are the
// algorithmic (not measured) HBM bytes and floating-point operations of the launch.
struct ProfScope {
  rb_ctx* ctx;
  size_t idx = 0;
  bool on;
  ProfScope(rb_ctx* c, int cls, double bytes, double flops) : ctx(c), on(c->profiling) {
    if (!on) return;
    rb_ctx::ProfRec r{cls, nullptr, nullptr, bytes, flops};
    if (cudaEventCreate(&r.a) != cudaSuccess || cudaEventCreate(&r.b) != cudaSuccess) { on = false; return; }
    cudaEventRecord(r.a, c->stream);
    idx = c->prof.size();
    c->prof.push_back(r);
  }
  ~ProfScope() {
    if (on) cudaEventRecord(ctx->prof[idx].b, ctx->stream);
  }
};

// Internal launchers shared between api.cu and model.cu (defined next to their kernels).
int tmap_2d_bf16(rb_ctx* ctx, const void* base, int64_t rows, int64_t cols, int64_t ld, int box_rows, CUtensorMap* out);

struct GemmArgs {
  const void* x = nullptr;      // [M, K]
  const void* w = nullptr;      // [N, K]
  const void* w2 = nullptr;     // gated: up weights [N, K]
  const void* bias = nullptr;   // [N]
  const void* residual = nullptr;  // [M, N]
  void* out = nullptr;          // [M, N] (model dtype) or float partials [n_split][M][N]
  int64_t m = 0, n = 0, k = 0;
  int act = RB_ACT_NONE;
  const void* act_params = nullptr;  // RB_ACT_XIELU: its two numbers, model dtype
  int n_split = 1;              // > 1: write float partials, no epilogue
  bool partials = false;
  // Grouped form: the rows of x are shared out among `experts` weight matrices stacked in w (and w2), see rb_moe_gated and rb_moe_up.
  const int32_t *list = nullptr, *count = nullptr;
  int64_t cap = 0;
  int experts = 0, top = 1;
  bool up = false;      // the first of an expert's two products (gated or not): from listed rows to compact ones
  bool sorted = false;  // up: x is already in the order of the lists
  bool reduce = false;            // M <= 64: if K is split, sum the splits inside the kernel and apply the epilogue
};
int gemm_tc_bf16(rb_ctx* ctx, const GemmArgs& a);
constexpr int kMaxExperts = 256;
int gemm_tc_grouped(rb_ctx* ctx, const GemmArgs& a);
bool grouped_wants_sorted(int64_t rows, int top, int experts);
int gemm_tc_pick_splits(rb_ctx* ctx, int64_t m, int64_t n, int64_t k);
int gemm_reserve_scratch(rb_ctx* ctx, size_t bytes);
int gemm_simple(rb_ctx* ctx, const GemmArgs& a, int dtype);

// moe.cu: rb_split_append and rb_moe_route, in one launch at single-token steps (route NULL: the first alone)
struct SplitSpec {
  const void* src = nullptr;
  const float* acc = nullptr;
  int n_acc = 0;
  const void* bias = nullptr;
  int64_t src_ld = 0;
  int batch = 0, s_new = 0, q_heads = 0, kv_heads = 0, dim = 0, glu_size = 0;
  rb_kv_cache* cache = nullptr;
  int layer = 0;
  void *q_out = nullptr, *glu_out = nullptr;
  int64_t glu_ld = 0;
};
struct RouteSpec {
  const float* acc = nullptr;
  int n_acc = 0;
  int64_t acc_stride = 0, z_ld = 0;
  int experts = 0, top = 0, groups = 1, keep = 1;
  float scale = 1.f;
  rb_route_options o{};
  int dtype = RB_BF16;         // of o.correction
  float* weight = nullptr;
  int32_t *list = nullptr, *count = nullptr;
  int64_t cap = 0;
};
int split_and_route(rb_ctx* ctx, const SplitSpec& split, const RouteSpec* route, int dtype);
// mixer_kernels.cu: rb_add_then_norm, and the experts' row counters back to zero for the next layer
struct JoinSpec {
  const void* y = nullptr;
  const float* acc = nullptr;
  int n_acc = 0;
  const void* part = nullptr;
  const float* weight = nullptr;
  int top = 0;
  float mult = 1.f;
  const float* own = nullptr;   // weight per row of `own_x`, rows in the model dtype (may be `out`); part rows of weight 0 are not read then
  const void* own_x = nullptr;
  const void* gain = nullptr;
  float eps = 0.f;
  int64_t rows = 0;
  int width = 0, ld = 0;
  float* h = nullptr;
  void* out = nullptr;
  int32_t* zero = nullptr;
  int n_zero = 0;
};
int add_then_norm(rb_ctx* ctx, const JoinSpec& s, int dtype);

// sandwich.cu: rb_sandwich_join
struct SandwichSpec {
  const void* y = nullptr;
  const float* acc = nullptr;
  int n_acc = 0;
  const void* post_gain = nullptr;
  int groups = 1;
  float eps = 0.f;
  int64_t rows = 0;
  int width = 0, ld = 0;
  const float* h_in = nullptr;
  float* h_out = nullptr;
  const void* depth = nullptr;
  int n_depth = 0;
  float* history = nullptr;
  int64_t history_stride = 0;
  const void* gain = nullptr;
  void* out = nullptr;
};
int sandwich_join(rb_ctx* ctx, const SandwichSpec& s, int dtype);

// What an attention layer may have beyond the plain causal form.
struct AttnExtra {
  int window = 0;              // rolling window: how many keys, its own included, a row sees; 0 = all
  int chunk = 0;               // > 0: a row sees only the keys of its own stretch of that many positions
  bool alibi = false;          // distance bias: 2^(-8 (h + 1) / q_heads) * (i - j) off the score of head h
  const void* gate = nullptr;  // out *= sigmoid(gate), model dtype, row pitch gate_ld
  int64_t gate_ld = 0;
  bool head_gate = false;      // gate has one number per head
  float out_scale = 1.f;       // factor on the output
  int value_dim = 0;           // columns of a head that are stored (the cache may hold padded heads)
  int64_t out_ld = 0;          // row pitch of the output
  int temp_every = 0;          // > 0: scores of the row at position p grow by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1)
  float temp_coef = 0.f;
  float softcap = 0.f;         // > 0: score <- softcap tanh(score / softcap)
  const void* sink = nullptr;  // [q_heads], cache dtype: exp(sink) joins the softmax denominator
  const void* talk = nullptr;  // [q_heads][q_heads], cache dtype: score[h] <- sum_g talk[h][g] score[g] before the mask
  const float* talk_host = nullptr;   // the same numbers on the host, or NULL
};
// the earliest position that the row at position `pos` sees (window 2^30: no window; chunk 0: no chunks)
__host__ __device__ __forceinline__ int first_visible(int pos, int window, int chunk) {
  const int lo = pos - window + 1 > 0 ? pos - window + 1 : 0;
  const int start = chunk > 0 ? pos - pos % chunk : 0;
  return lo > start ? lo : start;
}
// factor on the scores of the row at position `pos`
__device__ __forceinline__ float query_temperature(int pos, int every, float coef) {
  return every > 0 ? fmaf(coef, logf((float)((pos + 1) / every + 1)), 1.0f) : 1.0f;
}
// tanh to about 1e-7 absolute from two special-function operations; saturates without a NaN
__device__ __forceinline__ float tanh_sfu(float x) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * 2.8853900817779268f));
  return 1.0f - __fdividef(2.0f, 1.0f + e);
}
// slope of the distance bias, 2^(-8 (h + 1) / heads)
__device__ __forceinline__ float alibi_slope(int head, int heads) { return exp2f(-8.0f * (float)(head + 1) / (float)heads); }

int attention_mma_bf16(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads,
                       float scale, void* out, const AttnExtra* ext = nullptr);
bool attention_mma_takes(const rb_kv_cache* c, int q_heads);
// decoder_kernels.cu: the tensor-parallel sum of a row-parallel product (split-K slabs + bias, or a finished bf16
// tensor `part`) over the exchange buffers, the residual add and the following norm, in one kernel.
// sum_out = h + sum over ranks; out = norm(sum_out) (out may be NULL).  `parity` alternates 0,1,0,1.. launch by launch.
int exchange_norm(rb_ctx* ctx, const TpPeers& tp, int parity, int kind, const void* h, const float* acc, int n_acc,
                  const void* acc_bias, const void* part, const void* w, const void* b, float eps, int64_t rows,
                  int64_t hidden, void* out, void* sum_out);
// decoder_kernels.cu: out[r, j] = act(sum_s part[s][r][j] + bias[j]) (* sum_s part[s][r][j + n_out] when gated)
int act_from_partials(rb_ctx* ctx, const float* part, int n_split, int64_t rows, int64_t n_all, int64_t n_out, bool gated,
                      const void* bias, int act, void* out, const void* act_params = nullptr);
// Single-token step with the RoPE / KV-append work folded into the decode attention kernel (bf16 caches,
// head sizes that are multiples of 64).  `attention_can_fuse_rope` says whether the shapes and pointers allow it.
bool attention_can_fuse_rope(const rb_kv_cache* c, int q_heads, int rot, const void* qkv, const float* acc, int n_acc,
                             const void* bias, const float* cos_t, const float* sin_t, int batch);
int attention_decode_fused_rope(rb_ctx* ctx, const void* qkv, const float* acc, int n_acc, const void* bias,
                                const float* cos_t, const float* sin_t, int rot, rb_kv_cache* c, int layer, int batch,
                                int q_heads, float scale, void* out);
int attention_decode_splits(rb_ctx* ctx, int batch, int kv_heads, int max_len, int head_dim);
// keys a single-token step may have to walk under a rolling window or in chunks, for the split decision above
inline int attention_walk_len(int max_len, int window, int chunk = 0) {
  if (chunk > 0 && (window <= 0 || chunk < window)) window = chunk;
  return (window > 0 && window < max_len - 64) ? window + 64 : max_len;
}
int attention_reserve_scratch(rb_ctx* ctx, size_t bytes);
// attention_tc.cu: causal prefill attention on tcgen05 (head sizes 64 and 128, query length >= 128)
bool attention_prefill_tc_supported(const rb_kv_cache* c, int s_new, int q_heads, const void* q, const void* out);
int attention_prefill_tc(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads, float scale,
                         void* out, const AttnExtra* ext = nullptr);
// attention_latent.cu, attention_talk.cu: attention with mixed heads or over latents, one block for all heads of its tokens
bool attention_joint_takes(const rb_kv_cache* c, const AttnExtra& x);
int attention_joint_row_tiles(const rb_kv_cache* c, int q_heads);   // blocks a single token's heads take
int attention_joint(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads, float scale, void* out,
                    const AttnExtra& x);
// attention_mix_tc.cu: attention of prompts with mixed heads on tcgen05 (head sizes up to 128, up to 32 heads)
bool attention_mix_tc_takes(const rb_kv_cache* c, int s_new, int q_heads, const void* q, const AttnExtra& x);
int attention_mix_tc(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads, float scale, void* out,
                     const AttnExtra& x);
// plain_kernels.cu: attention whose heads' scores are mixed (x.talk), any sizes
int attention_talk_simple(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads, float scale, void* out,
                          int dtype, const AttnExtra& x);
int attention_simple(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads,
                     float scale, void* out, int dtype, const AttnExtra* ext = nullptr);
}  // namespace rb
