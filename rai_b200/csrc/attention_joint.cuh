// Attention in which one block has every head of its tokens, over the paged bf16 cache: heads whose scores are mixed before the
// softmax (score[h] <- sum_g talk[h][g] score[g]), and latent attention, where all heads read one wide vector per token that
// serves as key and, up to the latent's size, as value.  Prompts, portions of them and single tokens run the same kernel.
//
// Eight consumer warps and one that issues tiled copies.  Per tile of KT keys:
//   1  scores, transposed: S^T[keys x rows] = K . Q^T on mma.sync, a row being a (token, query head) that reads the tile's
//      key/value head; keys fill the 16-row side, so a single token's few heads waste nothing.  Raw scores go to shared memory.
//   2  a warp takes a few heads of a token (or a few rows): lanes are keys.  It mixes the raw scores of all heads (float32),
//      masks, and turns them into weights against a reference point that follows the running maximum lazily; weights go to
//      shared memory in bf16, the sum of a row stays in float32.
//   3  O^T[dims x rows] += V^T . P^T, accumulators in registers for the whole walk.
// The eight warps form teams of WG; a team has every TEAMS-th key/value head and reads only that head's tiles.  Inside a team the
// warps share out the dimensions of V, and for K two key halves times parts of the dot product (partial scores add in step 2).
// Copies run ahead through a ring of tiles: K of every head, then V of every head, and so on.
//
// Every wait is bounded; after a give-up the block runs on without waiting, writes nothing, reports, lets its copies land and
// returns.
#pragma once
#include <algorithm>
#include <vector>

#include "ctx.h"
#include "mma.cuh"
#include "ptx.cuh"

namespace rb {

using bf16 = __nv_bfloat16;

namespace joint {

constexpr float kLog2e = 1.4426950408889634f;
// Two warpgroups of consumers and one for the copies, which hands its registers over: 384 x 168 = 256 x 232 + 128 x 40.
constexpr int kConsumers = 256, kThreads = 384;
constexpr int kMaxStages = 24;
constexpr int kMaxSplits = 32;

struct Params {
  const bf16* q;               // [tokens][q_heads][D]
  const int32_t *block_table, *seq_lens;
  int pages_per_seq, s_new, D, q_heads, kv_heads, group;
  int row_tiles, tile_rows;    // rows (token, head of a key/value head) of a block: tile_rows <= 8 NT
  int nbk, nbv;                // 64-column blocks of a key and of a value that matter
  int stages, stage_bytes;
  int ring, own_rings;         // stages of a ring; whether each team has a ring of its own
  uint32_t ring_inv;           // ceil(2^32 / ring)
  int n_splits;
  int window, chunk, value_dim;
  float scale_log2;
  const bf16 *talk, *sink;
  bf16* out;
  int64_t out_ld;
  float *part_o, *part_ml;
  uint32_t *split_count, *status;
  long long wait_cycles;
};

// LATENT: one key/value head whose keys are the values, nothing mixed
template <int KT_, int WG_, int GP_, int DW_, int NT_, bool LATENT_>
struct Shape {
  static constexpr int KT = KT_, WG = WG_, GP = GP_, DW = DW_, NT = NT_;
  static constexpr bool LATENT = LATENT_;
  static constexpr int TEAMS = 8 / WG;
  static constexpr int SM = WG < 2 ? 1 : 2, SK = WG / SM;     // key halves, parts of the dot product
  static constexpr int MK = KT / 16 / SM;                     // 16-key tiles of a warp
  static constexpr int R = 8 * NT;                            // rows per key/value head
  static constexpr int SP = KT + 4, PP = KT + 8;              // pitches of scores (floats) and weights (bf16)
  static constexpr int KL = KT / 32;                          // keys per lane
  static constexpr int CH = NT == 1 ? 2 : 8;                  // heads that a warp mixes at a time
};

struct Layout {   // byte offsets behind the ring
  size_t q, s, p, talk, row, m, total;
};
template <typename S>
__host__ __device__ inline Layout layout_of(int G, int H, int nbk) {
  Layout l;
  size_t at = 0;
  const size_t rows = (size_t)G * S::R;
  l.q = at; at += rows * (nbk * 64 + 8) * 2;
  l.s = at; at += (size_t)S::SK * rows * S::SP * 4;
  l.p = at; at += rows * S::PP * 2;
  l.talk = at; at += S::LATENT ? 0 : (size_t)H * ((H + 7) / 8 * 8) * 4;
  l.row = at; at += S::LATENT ? 0 : (size_t)H * 4;
  l.m = at; at += rows * 3 * 4;
  l.total = at;
  return l;
}

__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(reinterpret_cast<unsigned long long&>(r))
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)),
        "l"(reinterpret_cast<unsigned long long&>(c)));
  return r;
}
__device__ __forceinline__ void ldsm_x2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void take_registers() { asm volatile("setmaxnreg.inc.sync.aligned.u32 232;"); }
__device__ __forceinline__ void give_registers() { asm volatile("setmaxnreg.dec.sync.aligned.u32 40;"); }
__device__ __forceinline__ void consumers_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// byte offset of the 16-byte chunk with (key, dims dc..dc+8) in a tile of column blocks [KT keys][128 bytes], 128-byte swizzle
template <int KT>
__device__ __forceinline__ int tile_off(int key, int dc) {
  return (dc >> 6) * (KT * 128) + key * 128 + ((((dc & 63) >> 3) ^ (key & 7)) << 4);
}

// Merges the splits of a single token's rows (the consumer warps; w_s: [row][split] weights over the row's sum)
template <typename S>
__device__ __forceinline__ void merge_splits(const Params& p, float* w_s, int b, int r0, int n_rows) {
  const int H = p.q_heads, vd = p.value_dim, ns = p.n_splits;
  const int live = S::LATENT ? n_rows : H;   // heads of the tile, or of the token
  auto head_of = [&](int i) { return S::LATENT ? (r0 + i) % p.group : i; };
  for (int i = threadIdx.x; i < live; i += kConsumers) {
    const int head = head_of(i);
    const float* ml = p.part_ml + ((size_t)b * H + head) * ns * 2;
    float M = -INFINITY, L = 0.f;
#pragma unroll 4
    for (int s = 0; s < ns; ++s) M = fmaxf(M, __ldcg(ml + 2 * s));
#pragma unroll 4
    for (int s = 0; s < ns; ++s) {
      const float w = ex2_fast(__ldcg(ml + 2 * s) - M);
      L = fmaf(w, __ldcg(ml + 2 * s + 1), L);
      w_s[i * kMaxSplits + s] = w;
    }
    if (p.sink) L += ex2_fast(fmaf(__bfloat162float(p.sink[head]), kLog2e, -M));
    const float inv = 1.0f / L;
    for (int s = 0; s < ns; ++s) w_s[i * kMaxSplits + s] *= inv;
  }
  consumers_sync();
  if ((vd & 3) == 0) {
    const int quads = vd >> 2;
#pragma unroll 2
    for (int i = threadIdx.x; i < live * quads; i += kConsumers) {
      const int row = i / quads, dim = (i - row * quads) * 4, head = head_of(row);
      const float4* src = reinterpret_cast<const float4*>(p.part_o + ((size_t)b * H + head) * ns * vd + dim);
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int s0 = 0; s0 < ns; s0 += 4) {
        float4 t[4];
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (s0 + k < ns) t[k] = __ldcg(src + (size_t)(s0 + k) * quads);
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (s0 + k < ns) {
            const float w = w_s[row * kMaxSplits + s0 + k];
            v.x = fmaf(t[k].x, w, v.x); v.y = fmaf(t[k].y, w, v.y); v.z = fmaf(t[k].z, w, v.z); v.w = fmaf(t[k].w, w, v.w);
          }
      }
      const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
      *reinterpret_cast<uint2*>(p.out + (size_t)b * p.out_ld + (size_t)head * vd + dim) =
          make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    }
    return;
  }
  for (int i = threadIdx.x; i < live * vd; i += kConsumers) {
    const int row = i / vd, dim = i % vd, head = head_of(row);
    const float* src = p.part_o + ((size_t)b * H + head) * ns * vd + dim;
    float v = 0.f;
    for (int sp = 0; sp < ns; ++sp) v = fmaf(__ldcg(src + (size_t)sp * vd), w_s[row * kMaxSplits + sp], v);
    p.out[(size_t)b * p.out_ld + (size_t)head * vd + dim] = __float2bfloat16_rn(v);
  }
}

template <typename S>
__global__ void __launch_bounds__(kThreads, 1) joint_attention_kernel(const Params p, const __grid_constant__ CUtensorMap tm_k,
                                                                      const __grid_constant__ CUtensorMap tm_v) {
  constexpr int KT = S::KT, NT = S::NT, R = S::R, GP = S::GP, DW = S::DW, SP = S::SP, PP = S::PP, KL = S::KL;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t full_bar[kMaxStages];
  __shared__ __align__(8) uint64_t empty_bar[kMaxStages];
  __shared__ volatile uint32_t abort_flag;
  __shared__ volatile int rescale_flag[2];
  __shared__ uint32_t full_turn[kMaxStages], is_last;   // copies issued into each stage
  uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int G = p.kv_heads, H = p.q_heads, group = p.group;
  const Layout lay = layout_of<S>(G, H, p.nbk);
  uint8_t* rest = ring + (size_t)p.stages * p.stage_bytes;
  bf16* q_s = reinterpret_cast<bf16*>(rest + lay.q);
  float* s_s = reinterpret_cast<float*>(rest + lay.s);
  bf16* p_s = reinterpret_cast<bf16*>(rest + lay.p);
  float* t_s = reinterpret_cast<float*>(rest + lay.talk);     // [g][h]: scale * log2(e) * talk[h][g]
  int* row_s = reinterpret_cast<int*>(rest + lay.row);        // first row of a head
  float* m_s = reinterpret_cast<float*>(rest + lay.m);        // reference point, sum, rescaling factor per row
  const int rows = G * R, qp = p.nbk * 64 + 8, hp = (H + 7) / 8 * 8;
  float* l_s = m_s + rows;
  float* c_s = l_s + rows;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    for (int s = 0; s < p.stages; ++s) { ptx::mbar_init(&full_bar[s], 1); ptx::mbar_init(&empty_bar[s], S::WG); }
    abort_flag = 0;
    rescale_flag[0] = rescale_flag[1] = 0;
    for (int s = 0; s < p.stages; ++s) full_turn[s] = 0;
    ptx::fence_barrier_init();
    ptx::fence_proxy_async();
    ptx::tma_prefetch_desc(&tm_k);
    if (!S::LATENT) ptx::tma_prefetch_desc(&tm_v);
  }
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait();   // q, lengths and the newest keys come from kernels before this one

  const int split = blockIdx.x, b = blockIdx.z;
  const int tile_row = p.s_new > 1 ? (int)gridDim.y - 1 - (int)blockIdx.y : (int)blockIdx.y;   // longest walks first
  const int r0 = tile_row * p.tile_rows, total_rows = p.s_new * group;
  const int n_rows = min(p.tile_rows, total_rows - r0);
  const int len = p.seq_lens[b], base = len - p.s_new;
  const int first_token = r0 / group, last_token = (r0 + n_rows - 1) / group;
  int tile_lo = first_visible(base + first_token, p.window, p.chunk) / KT;
  int tile_hi = (min(base + last_token + 1, len) + KT - 1) / KT;
  if (p.n_splits > 1) {
    const int per = (tile_hi - tile_lo + p.n_splits - 1) / p.n_splits;
    tile_lo += split * per;
    tile_hi = min(tile_hi, tile_lo + per);
  }
  const int units = S::LATENT ? 1 : 2 * G;   // copies per key tile
  // Stage of the copy of head g's keys or values of the it-th tile, and how often the stage has been used before.  One ring serves
  // all heads if it holds a tile of each: a team then never waits for a copy into a stage whose earlier copy, another
  // team's, may still be on its way (it would take that one for its own).  Otherwise each team has a ring of its own.
  auto place = [&](int it, int g, bool values, uint32_t& st) -> uint32_t {
    uint32_t u, first = 0;
    if (!p.own_rings) {
      u = (uint32_t)it * units + (values ? G + g : g);
    } else {
      const int t = g % S::TEAMS, heads = (G - t + S::TEAMS - 1) / S::TEAMS, a = g / S::TEAMS;
      u = (uint32_t)it * (2 * heads) + (values ? heads + a : a);
      first = t * p.ring;
    }
    const uint32_t turn = p.ring == 1 ? u : __umulhi(u, p.ring_inv);   // u / ring (u < 2^20)
    st = first + u - turn * p.ring;
    return turn;
  };

  if (warp >= 8) {
    // ------------------------------------------------------------------ copies
    give_registers();
    if (warp == 8 && lane == 0) {
      bool ok = true;
      for (int tile = tile_lo; tile < tile_hi && ok; ++tile) {
        const int page = p.block_table[(size_t)b * p.pages_per_seq + tile * KT / kPageTokens];
        for (int i = 0; i < units && ok; ++i) {
          uint32_t st;
          const uint32_t turn = place(tile - tile_lo, i < G ? i : i - G, i >= G, st);
          if (!ptx::mbar_wait(&empty_bar[st], (turn & 1u) ^ 1u, &abort_flag, p.wait_cycles)) { ok = false; break; }
          const bool v = i >= G;
          const int nb = v ? p.nbv : p.nbk, y = (page * G + (v ? i - G : i)) * kPageTokens + tile * KT % kPageTokens;
          ptx::mbar_expect_tx(&full_bar[st], (uint32_t)nb * KT * 128);
          for (int cb = 0; cb < nb; ++cb)
            ptx::tma_load_2d(ring + (size_t)st * p.stage_bytes + cb * (KT * 128), v ? &tm_v : &tm_k, &full_bar[st], cb * 64, y);
          full_turn[st] = turn + 1;
        }
      }
    }
  } else {
    // ------------------------------------------------------------------ what the walk starts from
    take_registers();
    float o[GP][DW][NT][4];
    for (int i = threadIdx.x; i < rows * (p.nbk * 8); i += kConsumers) {
      const int row = i / (p.nbk * 8), c = i % (p.nbk * 8) * 8, g = row / R, n = row % R;
      bf16* dst = q_s + (size_t)row * qp + c;
      if (n < n_rows) {
        const int token = p.s_new == 1 ? 0 : (r0 + n) / group, head = g * group + r0 + n - token * group;
        cp_async16(dst, p.q + (((size_t)b * p.s_new + token) * H + head) * p.D + c);
      } else {
        *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
      }
    }
    cp_async_commit();
    for (int i = threadIdx.x; i < rows * (PP / 8); i += kConsumers) reinterpret_cast<uint4*>(p_s)[i] = make_uint4(0, 0, 0, 0);
    for (int i = threadIdx.x; i < rows; i += kConsumers) { m_s[i] = -INFINITY; l_s[i] = 0.f; c_s[i] = 1.f; }
    if (!S::LATENT)
      for (int h = threadIdx.x; h < H; h += kConsumers) row_s[h] = h / group * R + h % group;
    if (!S::LATENT) {
#pragma unroll 4
      for (int i = threadIdx.x; i < H * hp; i += kConsumers) {
        const int h = i / H, g = i - h * H;   // (neighbouring threads read neighbours)
        t_s[g * hp + h] = h < H ? __bfloat162float(__ldg(p.talk + min(i, H * H - 1))) * p.scale_log2 : 0.f;
      }
    }
    cp_async_wait<0>();
    consumers_sync();
#pragma unroll
    for (int a = 0; a < GP; ++a)
#pragma unroll
      for (int d = 0; d < DW; ++d)
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[a][d][n][0] = o[a][d][n][1] = o[a][d][n][2] = o[a][d][n][3] = 0.f; }

    const int team = warp / S::WG, wi = warp % S::WG, g8 = lane >> 2, t4 = lane & 3;
    const int km = wi % S::SM, ks = wi / S::SM;
    const int steps = p.nbk * 4, per_part = (steps + S::SK - 1) / S::SK, k_lo = ks * per_part, k_hi = min(steps, k_lo + per_part);
    const int live_dims = p.value_dim, n_tokens = S::LATENT ? 1 : n_rows / group;
    const bool windowed = p.window < (1 << 30) || p.chunk > 0;
    bool rescaled = false;        // this warp's rows had other factors than 1 in the tile before
    float m_row[NT], l_row[NT];   // LATENT: of this warp's rows
    int seen_from[NT], seen_to[NT];
    if constexpr (S::LATENT) {
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int row = warp * NT + i;
        m_row[i] = -INFINITY;
        l_row[i] = 0.f;
        seen_to[i] = row < n_rows ? base + (r0 + row) / group : -1;
        seen_from[i] = row < n_rows ? first_visible(seen_to[i], p.window, p.chunk) : 0;
      }
    }
    for (int tile = tile_lo; tile < tile_hi; ++tile) {
      const int it = tile - tile_lo, key0 = tile * KT;
      // ---------------------------------------------------------------- 1: raw scores
#pragma unroll
      for (int a = 0; a < GP; ++a) {
        const int g = a * S::TEAMS + team;
        if (g >= G) continue;
        uint32_t st;
        const uint32_t turn = place(it, g, false, st);
        ptx::mbar_wait(&full_bar[st], turn & 1u, &abort_flag, p.wait_cycles);
        __syncwarp();
        const uint32_t kt = s_u32(ring + (size_t)st * p.stage_bytes);
        constexpr int NC = NT < 4 ? NT : 4;
#pragma unroll
        for (int nc = 0; nc < NT / NC; ++nc) {
          float s[S::MK][NC][4];
#pragma unroll
          for (int m = 0; m < S::MK; ++m)
#pragma unroll
            for (int n = 0; n < NC; ++n) { s[m][n][0] = s[m][n][1] = s[m][n][2] = s[m][n][3] = 0.f; }
          const uint32_t qa = s_u32(q_s + (size_t)(g * R + nc * NC * 8) * qp);
#pragma unroll 4
          for (int kk = k_lo; kk < k_hi; ++kk) {
            uint32_t af[S::MK][4];
#pragma unroll
            for (int m = 0; m < S::MK; ++m)
              ldsm_x4(af[m], kt + tile_off<KT>(km * (KT / S::SM) + m * 16 + (lane & 15), kk * 16 + (lane >> 4) * 8));
            if constexpr (NC == 1) {
              uint32_t b0, b1;
              ldsm_x2(b0, b1, qa + (uint32_t)(((lane & 7) * qp + kk * 16 + ((lane >> 3) & 1) * 8) * 2));
#pragma unroll
              for (int m = 0; m < S::MK; ++m) mma16816(s[m][0], af[m], b0, b1);
            } else {
#pragma unroll
              for (int j = 0; j < NC / 2; ++j) {
                uint32_t bf[4];
                ldsm_x4(bf, qa + (uint32_t)(((j * 16 + (lane & 7) + ((lane >> 4) << 3)) * qp + kk * 16 + ((lane >> 3) & 1) * 8) * 2));
#pragma unroll
                for (int m = 0; m < S::MK; ++m) { mma16816(s[m][2 * j], af[m], bf[0], bf[1]); mma16816(s[m][2 * j + 1], af[m], bf[2], bf[3]); }
              }
            }
          }
          float* dst = s_s + ((size_t)ks * rows + g * R + nc * NC * 8) * SP + km * (KT / S::SM);
#pragma unroll
          for (int m = 0; m < S::MK; ++m)
#pragma unroll
            for (int n = 0; n < NC; ++n)
#pragma unroll
              for (int e = 0; e < 4; ++e) dst[(n * 8 + 2 * t4 + (e & 1)) * SP + m * 16 + g8 + (e >> 1) * 8] = s[m][n][e];
        }
        if (!S::LATENT) {
          __syncwarp();
          if (lane == 0) ptx::mbar_arrive(&empty_bar[st]);
        }
      }
      consumers_sync();
      // ---------------------------------------------------------------- 2: mixing, mask, weights
      if (threadIdx.x == 0) rescale_flag[(it + 1) & 1] = 0;
      auto raw = [&](int row, float (&v)[KL]) {   // the parts of the dot product added up
#pragma unroll
        for (int e = 0; e < KL; ++e) v[e] = 0.f;
#pragma unroll
        for (int k = 0; k < S::SK; ++k) {
          const float* src = s_s + ((size_t)k * rows + row) * SP + lane * KL;
          if constexpr (KL == 1) v[0] += src[0];
          else { const float2 t = *reinterpret_cast<const float2*>(src); v[0] += t.x; v[KL - 1] += t.y; }
        }
      };
      auto store_weights = [&](int row, const float (&v)[KL]) {
        bf16* dst = p_s + (size_t)row * PP + lane * KL;
        if constexpr (KL == 1) dst[0] = __float2bfloat16_rn(v[0]);
        else *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(v[0], v[KL - 1]);
      };
      if constexpr (S::LATENT) {   // a warp has NT rows for the whole walk: reference points and sums stay in registers
        float v[NT][KL], top[NT];
#pragma unroll
        for (int i = 0; i < NT; ++i) raw(warp * NT + i, v[i]);
        const bool edge = key0 + KT - 1 > base + first_token || windowed;   // a key that some row does not see
        bool outgrown = false;
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          top[i] = -INFINITY;
#pragma unroll
          for (int e = 0; e < KL; ++e) {
            v[i][e] *= p.scale_log2;
            const int k = key0 + lane * KL + e;
            if (edge && (k > seen_to[i] || k < seen_from[i])) v[i][e] = -INFINITY;
            top[i] = fmaxf(top[i], v[i][e]);
          }
          outgrown |= top[i] > m_row[i] + 8.0f;   // the reference point moves only when the maximum has outgrown it by 2^8
        }
        if (rescaled) {   // (the factors of the tile before have been read)
          if (lane == 0)
            for (int i = 0; i < NT; ++i) c_s[warp * NT + i] = 1.f;
          rescaled = false;
        }
        if (__any_sync(0xffffffffu, outgrown)) {
#pragma unroll
          for (int i = 0; i < NT; ++i) {
            const float best = warp_max(top[i]);
            if (best > m_row[i] + 8.0f) {
              const float c = ex2_fast(m_row[i] - best);
              l_row[i] *= c;
              if (lane == 0) {
                c_s[warp * NT + i] = c;
                if (m_row[i] != -INFINITY) rescale_flag[it & 1] = 1;
              }
              m_row[i] = best;
            }
          }
          rescaled = true;
        }
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          const float use = m_row[i] == -INFINITY ? 0.f : m_row[i];
#pragma unroll
          for (int e = 0; e < KL; ++e) { v[i][e] = ex2_fast(v[i][e] - use); l_row[i] += v[i][e]; }
          store_weights(warp * NT + i, v[i]);
        }
      } else {
        constexpr int CH = S::CH;
        const int chunks = (H + CH - 1) / CH, n_units = chunks * n_tokens;
        const bool any_factors = rescaled;
        bool any_moved = false;
        for (int unit = warp; unit < n_units; unit += 8) {
          const int tok = n_tokens == 1 ? 0 : unit / chunks, h0 = (unit - tok * chunks) * CH;
          float2 acc[CH / 2][KL];
#pragma unroll
          for (int i = 0; i < CH / 2; ++i)
#pragma unroll
            for (int e = 0; e < KL; ++e) acc[i][e] = make_float2(0.f, 0.f);
          constexpr int B = CH == 8 ? 4 : 8;   // raw heads in flight
          for (int g0 = 0; g0 < H; g0 += B) {
            float x[B][KL];
            float2 t2[B][CH / 2];
#pragma unroll
            for (int g = 0; g < B; ++g) {
              const int gg = min(g0 + g, H - 1);
              raw(row_s[gg] + tok * group, x[g]);
#pragma unroll
              for (int i = 0; i < CH / 2; ++i) t2[g][i] = *reinterpret_cast<const float2*>(t_s + gg * hp + h0 + 2 * i);
            }
#pragma unroll
            for (int g = 0; g < B; ++g)
              if (g0 + g < H) {
#pragma unroll
                for (int i = 0; i < CH / 2; ++i)
#pragma unroll
                  for (int e = 0; e < KL; ++e) acc[i][e] = fma2(t2[g][i], make_float2(x[g][e], x[g][e]), acc[i][e]);
              }
          }
          const int seen_hi = base + r0 / group + tok, seen_lo = first_visible(seen_hi, p.window, p.chunk);
          float sum[CH], m[CH], v[CH][KL], top[CH];
          int at[CH];
          bool outgrown = false;
#pragma unroll
          for (int i = 0; i < CH; ++i) {
            at[i] = row_s[min(h0 + i, H - 1)] + tok * group;
            m[i] = m_s[at[i]];
          }
#pragma unroll
          for (int i = 0; i < CH; ++i) {
            top[i] = -INFINITY;
#pragma unroll
            for (int e = 0; e < KL; ++e) {
              const int key = key0 + lane * KL + e;
              const float x = (i & 1) ? acc[i >> 1][e].y : acc[i >> 1][e].x;
              v[i][e] = key <= seen_hi && key >= seen_lo ? x : -INFINITY;
              top[i] = fmaxf(top[i], v[i][e]);
            }
            outgrown |= h0 + i < H && top[i] > m[i] + 8.0f;   // the reference point moves only when the maximum has outgrown it by 2^8
          }
          const bool moves = __any_sync(0xffffffffu, outgrown);
          if (moves || any_factors) {   // (factors other than 1 of the tile before have been read)
#pragma unroll
            for (int i = 0; i < CH; ++i) {
              const float best = moves ? warp_max(top[i]) : -INFINITY, old = m[i];
              const bool move = best > old + 8.0f;
              if (move) m[i] = best;
              __syncwarp();
              if (lane == 0 && h0 + i < H) {
                const float c = move ? ex2_fast(old - best) : 1.f;
                c_s[at[i]] = c;
                m_s[at[i]] = m[i];
                l_s[at[i]] *= c;
                if (move && old != -INFINITY) rescale_flag[it & 1] = 1;
              }
            }
            any_moved |= moves;
          }
#pragma unroll
          for (int i = 0; i < CH; ++i) {
            sum[i] = 0.f;
            if (h0 + i >= H) continue;
            const float use = m[i] == -INFINITY ? 0.f : m[i];
#pragma unroll
            for (int e = 0; e < KL; ++e) { v[i][e] = ex2_fast(v[i][e] - use); sum[i] += v[i][e]; }
            store_weights(at[i], v[i]);
          }
          if constexpr (CH == 8) {   // eight sums over the lanes at once; lane 4 i ends up with the i-th
#pragma unroll
            for (int half = 4; half >= 1; half >>= 1)
#pragma unroll
              for (int i = 0; i < half; ++i) {
                const bool up = lane & (half * 4);
                const float keep = up ? sum[i + half] : sum[i], send = up ? sum[i] : sum[i + half];
                sum[i] = keep + __shfl_xor_sync(0xffffffffu, send, half * 4);
              }
            sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], 2);
            sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], 1);
            __syncwarp();   // (lane 0 may have rescaled a row's sum)
            if ((lane & 3) == 0 && h0 + (lane >> 2) < H) l_s[row_s[h0 + (lane >> 2)] + tok * group] += sum[0];
            __syncwarp();
          } else {
#pragma unroll
            for (int i = 0; i < CH; ++i) sum[i] = warp_sum(sum[i]);
            if (lane == 0)
              for (int i = 0; i < CH; ++i)
                if (h0 + i < H) l_s[at[i]] += sum[i];
          }
        }
        rescaled = any_moved;
      }
      consumers_sync();
      // ---------------------------------------------------------------- 3: values
      const bool rescale = rescale_flag[it & 1] != 0;
#pragma unroll
      for (int a = 0; a < GP; ++a) {
        const int g = a * S::TEAMS + team;
        if (g >= G) continue;
        uint32_t st;
        const uint32_t turn = place(it, g, !S::LATENT, st);
        if (!S::LATENT) {
          ptx::mbar_wait(&full_bar[st], turn & 1u, &abort_flag, p.wait_cycles);
          __syncwarp();
        }
        const uint32_t vt = s_u32(ring + (size_t)st * p.stage_bytes);
        if (rescale) {
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            const float c0 = c_s[g * R + n * 8 + 2 * t4], c1 = c_s[g * R + n * 8 + 2 * t4 + 1];
#pragma unroll
            for (int d = 0; d < DW; ++d) { o[a][d][n][0] *= c0; o[a][d][n][1] *= c1; o[a][d][n][2] *= c0; o[a][d][n][3] *= c1; }
          }
        }
#pragma unroll
        for (int k2 = 0; k2 < KL; ++k2) {
          uint32_t pf[NT][4];   // weights of 32 keys
#pragma unroll
          for (int n = 0; n < NT; ++n)
            ldsm_x4(pf[n], s_u32(p_s + (size_t)(g * R + n * 8 + (lane & 7)) * PP + k2 * 32 + (lane >> 3) * 8));
#pragma unroll
          for (int d = 0; d < DW; ++d) {
            const int dim0 = (wi * DW + d) * 16;
            if (dim0 >= live_dims) continue;
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
              uint32_t af[4];
              ldsm_x4_t(af, vt + tile_off<KT>(k2 * 32 + hf * 16 + (lane & 7) + ((lane >> 4) << 3), dim0 + ((lane >> 3) & 1) * 8));
#pragma unroll
              for (int n = 0; n < NT; ++n) mma16816(o[a][d][n], af, pf[n][2 * hf], pf[n][2 * hf + 1]);
            }
          }
        }
        __syncwarp();
        if (lane == 0) ptx::mbar_arrive(&empty_bar[st]);
      }
    }
    if constexpr (S::LATENT) {
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const float l = warp_sum(l_row[i]);
        if (lane == 0) { m_s[warp * NT + i] = m_row[i]; l_s[warp * NT + i] = l; }
      }
    }
    consumers_sync();
    if (!abort_flag) {
      // ---------------------------------------------------------------- output
      const int vd = p.value_dim, ns = p.n_splits;
#pragma unroll
      for (int a = 0; a < GP; ++a) {
        const int g = a * S::TEAMS + team;
        if (g >= G) continue;
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e2 = 0; e2 < 2; ++e2) {
            const int row = n * 8 + 2 * t4 + e2;
            if (row >= n_rows) continue;
            const int token = (r0 + row) / group, head = g * group + (r0 + row) % group;
            const float m = m_s[g * R + row];
            float l = l_s[g * R + row];
            if (ns == 1) {
              if (p.sink) l += ex2_fast(fmaf(__bfloat162float(p.sink[head]), kLog2e, -m));
              const float inv = 1.0f / l;
              bf16* dst = p.out + ((size_t)b * p.s_new + token) * p.out_ld + (size_t)head * vd;
#pragma unroll
              for (int d = 0; d < DW; ++d) {
                const int dim = (wi * DW + d) * 16 + g8;
                if (dim < vd) dst[dim] = __float2bfloat16_rn(o[a][d][n][e2] * inv);
                if (dim + 8 < vd) dst[dim + 8] = __float2bfloat16_rn(o[a][d][n][2 + e2] * inv);
              }
            } else {
              const size_t at = ((size_t)b * H + head) * ns + split;   // (single tokens)
#pragma unroll
              for (int d = 0; d < DW; ++d) {
                const int dim = (wi * DW + d) * 16 + g8;
                if (dim < vd) p.part_o[at * vd + dim] = o[a][d][n][e2];
                if (dim + 8 < vd) p.part_o[at * vd + dim + 8] = o[a][d][n][2 + e2];
              }
              if (wi == 0 && g8 == 0) { p.part_ml[at * 2] = m; p.part_ml[at * 2 + 1] = l; }
            }
          }
      }
      if (ns > 1) {
        // The block that arrives last for these rows merges all splits, in split order.
        __threadfence();
        consumers_sync();
        if (threadIdx.x == 0) {
          uint32_t* cnt = p.split_count + (size_t)b * p.row_tiles + tile_row;
          is_last = atomicAdd(cnt, 1u) == (uint32_t)ns - 1u ? 1u : 0u;
          if (is_last) *cnt = 0u;   // re-armed for the next launch
          __threadfence();
        }
        consumers_sync();
        if (is_last) merge_splits<S>(p, reinterpret_cast<float*>(ring), b, r0, n_rows);
      }
    }
  }
  __syncthreads();
  if (abort_flag && threadIdx.x == 0) {
    p.status[0] = (uint32_t)(-RB_ERR_TIMEOUT); p.status[1] = 0xA701u; p.status[2] = blockIdx.y; p.status[3] = blockIdx.z;
    volatile uint32_t never = 0;   // copies already on their way get a bounded chance to land
    for (int st = 0; st < p.stages; ++st)
      if (full_turn[st] > 0) ptx::mbar_wait(&full_bar[st], (full_turn[st] - 1u) & 1u, &never, p.wait_cycles);
  }
}

constexpr size_t kSmemLimit = 227 * 1024 - 4096;   // (the static part and alignment)

// Ring depth that fits; 0: not even two tiles do
template <typename S>
int ring_of(const Params& p, size_t* bytes) {
  const Layout l = layout_of<S>(p.kv_heads, p.q_heads, p.nbk);
  if (l.total + 2 * (size_t)p.stage_bytes > kSmemLimit) return 0;
  const int stages = (int)std::min<size_t>({(size_t)kMaxStages, (kSmemLimit - l.total) / p.stage_bytes, (size_t)std::max(3, 2 * 96 * 1024 / p.stage_bytes)});
  *bytes = l.total + (size_t)stages * p.stage_bytes + 1024;
  return stages;
}

// RB_ERR_UNIMPLEMENTED (without an error text): this shape does not fit
template <typename S>
int launch(rb_ctx* ctx, rb_kv_cache* c, Params p, int layer, int batch, int max_len) {
  p.stage_bytes = S::KT * 128 * std::max(p.nbk, S::LATENT ? 0 : p.nbv);
  size_t smem = 0;
  p.stages = ring_of<S>(p, &smem);
  const int whole = p.s_new * p.group;
  p.own_rings = !S::LATENT && p.stages < p.kv_heads;
  p.ring = p.own_rings ? p.stages / S::TEAMS : p.stages;
  if (p.ring == 0) return RB_ERR_UNIMPLEMENTED;
  p.ring_inv = (uint32_t)std::min<uint64_t>(0xffffffffull, ((1ull << 32) + p.ring - 1) / p.ring);
  p.tile_rows = std::min(whole, S::LATENT ? S::R : S::R / p.group * p.group);
  if (p.tile_rows == 0) return RB_ERR_UNIMPLEMENTED;
  p.row_tiles = (whole + p.tile_rows - 1) / p.tile_rows;
  p.n_splits = 1;
  if (p.s_new == 1 && p.row_tiles <= (S::LATENT ? ::kLatentRowTiles : 1)) {
    p.n_splits = attention_decode_splits(ctx, batch, p.row_tiles, max_len, 256);
    if (p.n_splits > kMaxSplits) p.n_splits = kMaxSplits;
    if (p.n_splits > 1) {
      const size_t parts = (size_t)batch * p.q_heads * p.n_splits;
      RB_TRY(attention_reserve_scratch(ctx, parts * (p.value_dim + 2) * sizeof(float)));
      p.part_o = ctx->attn_scratch;
      p.part_ml = ctx->attn_scratch + parts * p.value_dim;
    }
  }
  auto kern = joint_attention_kernel<S>;
  static size_t set[64] = {};
  const int dv = ctx->device & 63;
  if (smem > set[dv]) { RB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); set[dv] = smem; }
  CUtensorMap tk{}, tv{};
  const size_t off = (size_t)layer * c->layer_stride_elems();
  const int64_t rows = (int64_t)c->num_pages * c->kv_heads * kPageTokens;
  RB_TRY(tmap_2d_bf16(ctx, (const bf16*)c->k + off, rows, p.D, p.D, S::KT, &tk));
  if (!S::LATENT) RB_TRY(tmap_2d_bf16(ctx, (const bf16*)c->v + off, rows, p.D, p.D, S::KT, &tv));
  const dim3 grid((unsigned)p.n_splits, (unsigned)p.row_tiles, (unsigned)batch);
  if (grid.y > 65535) return RB_ERR_UNIMPLEMENTED;
  RB_CUDA(launch_kernel(kern, grid, dim3(kThreads), smem, ctx->stream, ctx->pdl, p, tk, tv));
  ctx->launches++;
  return RB_OK;
}

}  // namespace joint

}  // namespace rb
