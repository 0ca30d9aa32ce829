// Causal attention of prompts whose heads' scores are mixed before the softmax (score[h] <- sum_g talk[h][g] score[g]), on the
// 5th-generation tensor cores, for head sizes up to 128 and up to 32 heads over the paged bf16 cache.
//
// One CTA has MT = 256 / HP tokens with all their heads (HP: the number of heads rounded up to 8, 16 or 32), so that no raw score
// is computed twice.  Both products are transposed: keys, then dimensions, fill the 128 lanes of tensor memory, and a column is
// a (head, token):
//   S^T [128 keys x 256]  = K . Q^T      per key/value head: its heads' columns, K and Q K-major
//   O^T [128 dims x 256] += V^T . P^T    V and P MN-major, straight from their [keys][...] tiles
// which fills the 512 columns of tensor memory.  Twelve warps:
//   warps 0-7   a thread has one key (its lane) and 64 columns at a time, all heads of a few tokens: it reads the raw scores,
//               mixes them in float32 (packed FMAs), masks, and stores the weights in bf16.  The reference point of the
//               exponentials is one number per column for all 128 keys, 2^6 above the maximum when it was set.  A tile is
//               computed on the reference points as they are; only if a score has outgrown its own by 2 (always at the first
//               tile) do the warps set new ones and compute the tile again, from raw scores that the warp in question has
//               not given back.  The sums of the weights over the keys come from a product with ones on mma.sync, in
//               float32.
//   warp 8      tiled copies: Q once, then K of every head, V of every head, ... through a ring of 128-key tiles (two pages);
//   warp 9      owns the tensor memory; one lane issues the products: the scores of the next tile as soon as the raw scores of
//               this one have been read, so that they are there when its weights are done.
// Every wait is bounded; after a give-up the block runs on without waiting, writes nothing, reports, lets its copies land, frees its
// tensor memory and returns.
#include <algorithm>

#include "ctx.h"
#include "mma.cuh"
#include "ptx.cuh"

namespace rb {

using bf16 = __nv_bfloat16;

namespace {

constexpr int kKeys = 128;                   // keys per tile = lanes
constexpr int kThreads = 384;                // 384 x 168 = 256 x 232 + 128 x 40 registers
constexpr int kWarps = 8, kSoftmax = 256;
constexpr int kCols = 256;                   // columns of S and of O
constexpr int kBlock = kKeys * 128;          // 64 columns of 128 keys (or of P's rows), 128-byte swizzle; a stage of the ring
constexpr int kPageBlock = kPageTokens * 128;
constexpr int kMaxStages = 8;
constexpr float kLog2e = 1.4426950408889634f;

struct MixParams {
  const int32_t *block_table, *seq_lens;
  int pages_per_seq, s_new, q_heads, kv_heads, group, D, nb, nbv;
  int head_cols;              // columns of a key/value head: group * MT, rounded up so that no block of 64 is crossed
  int stages, value_dim;
  int column[32];             // of a head's first token
  const bf16* sink;
  bf16* out;
  int64_t out_ld;
  uint32_t* status;
  long long wait_cycles;
};

struct MixCtrl {
  uint64_t q_full, full[kMaxStages], empty[kMaxStages], s_full, s_empty, p_full, o_done;
  uint32_t tmem_base, abort_flag, issued, grow[2][2];   // grow: [half][tile & 1]
};

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(reinterpret_cast<unsigned long long&>(r))
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)),
        "l"(reinterpret_cast<unsigned long long&>(c)));
  return r;
}
__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// among the eight softmax warps, and among the four of a half
__device__ __forceinline__ void softmax_sync() {
  __syncwarp();
  asm volatile("bar.sync 1, 256;" ::: "memory");
}
template <bool kHalves>
__device__ __forceinline__ void half_sync(int half) {
  if (!kHalves) return softmax_sync();
  __syncwarp();
  asm volatile("bar.sync %0, 128;" ::"r"(2 + half) : "memory");
}
__device__ __forceinline__ float max3(float a, float b, float c) {
  float r;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c));
  return r;
}

template <int HP>
struct MixShape {
  static constexpr int MT = kCols / HP;      // tokens of a CTA
  static constexpr int TC = 64 / HP;         // tokens of a thread at a time
  // Warps 0-3 have the first half of the tokens, warps 4-7 the second.  Where eight neighbouring columns belong to one half, each
  // half goes its own way within a tile; otherwise all eight warps move together.
  static constexpr bool kHalves = MT >= 16;
  static __device__ __forceinline__ int eighth(int warp, int k) {   // the k-th of the four groups of 8 columns a warp adds up
    const int i = (warp & 3) * 4 + k;
    return !kHalves ? warp * 4 + k : i / (MT / 16) * (MT / 8) + (warp >> 2) * (MT / 16) + i % (MT / 16);
  }
  static __device__ __forceinline__ int own_column(int thread) {     // one column per thread, of its half
    const int i = thread & 127;
    return !kHalves ? thread : i / (MT / 2) * MT + (thread >> 7) * (MT / 2) + i % (MT / 2);
  }
  // behind Q, P and the ring: minus the reference points and their shifts, per column
  static constexpr size_t fixed_bytes(int nb) { return (size_t)nb * kCols * 128 + 4 * kBlock + 2 * kCols * 4 + sizeof(MixCtrl); }
};

// scale * log2(e) * talk[h][g], every number twice, as operands of the launch: constants to the mixing, which would otherwise spend
// more on fetching them from shared memory than on its multiply-adds
template <int HP>
struct MixTalk {
  float2 t[HP * HP];
};

template <int HP>
__global__ void __launch_bounds__(kThreads, 1) attention_mix_tc_kernel(const __grid_constant__ CUtensorMap tm_q,
                                                                      const __grid_constant__ CUtensorMap tm_k,
                                                                      const __grid_constant__ CUtensorMap tm_v, const MixParams p,
                                                                      const __grid_constant__ MixTalk<HP> talk) {
  using C = MixShape<HP>;
  constexpr int MT = C::MT, TC = C::TC;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* q_s = smem;                                                  // [nb][256 columns][128 bytes]
  uint8_t* p_s = q_s + (size_t)p.nb * kCols * 128;                      // [4][128 keys][128 bytes]
  uint8_t* ring = p_s + 4 * kBlock;
  float* m_s = reinterpret_cast<float*>(ring + (size_t)p.stages * kBlock);   // minus the reference point, per column
  float* shift_s = m_s + kCols;                                         // by how much it has just moved; at the end 1 / sum
  MixCtrl* ctl = reinterpret_cast<MixCtrl*>(shift_s + kCols);
  volatile uint32_t* abort_flag = &ctl->abort_flag;
  const int warp = __shfl_sync(0xffffffffu, (int)threadIdx.x >> 5, 0), lane = threadIdx.x & 31;   // (uniform, and seen to be)
  const int G = p.kv_heads, H = p.q_heads;

  if (threadIdx.x == 0) {
    ptx::mbar_init(&ctl->q_full, 1);
    for (int i = 0; i < p.stages; ++i) { ptx::mbar_init(&ctl->full[i], 1); ptx::mbar_init(&ctl->empty[i], 1); }
    ptx::mbar_init(&ctl->s_full, 1);
    ptx::mbar_init(&ctl->s_empty, kWarps);
    ptx::mbar_init(&ctl->p_full, kWarps);
    ptx::mbar_init(&ctl->o_done, 1);
    ctl->abort_flag = ctl->issued = 0;
    ctl->grow[0][0] = ctl->grow[0][1] = ctl->grow[1][0] = ctl->grow[1][1] = 0;
    ptx::fence_barrier_init();
    ptx::fence_proxy_async();
    ptx::tma_prefetch_desc(&tm_q);
    ptx::tma_prefetch_desc(&tm_k);
    ptx::tma_prefetch_desc(&tm_v);
  }
  if (warp == 9) {
    ptx::tmem_alloc(&ctl->tmem_base, 512);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tmem_s = ctl->tmem_base, tmem_o = tmem_s + kCols;
  pdl_launch_dependents();
  pdl_wait();   // q, lengths and the newest keys come from kernels before this one

  const int t0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * MT, b = blockIdx.y;   // longest walks first
  const int len = p.seq_lens[b], base = len - p.s_new;
  const int n = (min(base + t0 + MT, len) + kKeys - 1) / kKeys;                  // tiles
  // the swizzle atoms must sit on 1024-byte boundaries
  const bool layout_ok = (ptx::smem_u32(smem) & 1023u) == 0u && n >= 1;
  if (!layout_ok && threadIdx.x == 0) { p.status[0] = (uint32_t)(-RB_ERR_CUDA); p.status[1] = 0xA710u; p.status[2] = blockIdx.x; }

  if (warp >= 8) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 40;");
    if (layout_ok && warp == 8 && lane == 0) {
      // ------------------------------------------------------------------ copies
      ptx::mbar_expect_tx(&ctl->q_full, (uint32_t)(H * p.nb * MT * 128));
      for (int h = 0; h < H; ++h)
        for (int cb = 0; cb < p.nb; ++cb)
          ptx::tma_load_2d(q_s + (size_t)cb * kCols * 128 + (size_t)p.column[h] * 128, &tm_q, &ctl->q_full,
                           h * p.D + cb * 64, b * p.s_new + t0);
      uint32_t phase = 1u;
      int st = 0;
      bool ok = true;
      // a stage is 64 columns of a tile's keys, or one page of its values
      auto next_stage = [&](uint32_t bytes) -> uint8_t* {
        if (!ptx::mbar_wait(&ctl->empty[st], phase, abort_flag, p.wait_cycles)) { ok = false; return nullptr; }
        ptx::mbar_expect_tx(&ctl->full[st], bytes);
        return ring + (size_t)st * kBlock;
      };
      auto advance = [&]() {
        ++ctl->issued;
        if (++st == p.stages) { st = 0; phase ^= 1u; }
      };
      auto page_of = [&](int i) { return p.block_table[(size_t)b * p.pages_per_seq + min(i, p.pages_per_seq - 1)]; };
      auto load_keys = [&](int tile) {
        const int page0 = page_of(tile * 2), page1 = page_of(tile * 2 + 1);
        for (int g = 0; g < G; ++g)
          for (int cb = 0; cb < p.nb; ++cb) {
            uint8_t* dst = next_stage(kBlock);
            if (!dst) return;
            ptx::tma_load_2d(dst, &tm_k, &ctl->full[st], cb * 64, (page0 * G + g) * kPageTokens);
            ptx::tma_load_2d(dst + kPageBlock, &tm_k, &ctl->full[st], cb * 64, (page1 * G + g) * kPageTokens);
            advance();
          }
      };
      auto load_values = [&](int tile) {
        const int page[2] = {page_of(tile * 2), page_of(tile * 2 + 1)};
        for (int i = 0; i < G * 2; ++i) {
          const int y = (page[i & 1] * G + (i >> 1)) * kPageTokens;
          uint8_t* dst = next_stage((uint32_t)p.nbv * kPageBlock);
          if (!dst) return;
          for (int cb = 0; cb < p.nbv; ++cb) ptx::tma_load_2d(dst + cb * kPageBlock, &tm_v, &ctl->full[st], cb * 64, y);
          advance();
        }
      };
      load_keys(0);
      for (int j = 0; j < n && ok; ++j) {
        if (j + 1 < n) load_keys(j + 1);
        if (ok) load_values(j);
      }
    } else if (layout_ok && warp == 9 && lane == 0) {
      // ------------------------------------------------------------------ products
      const uint32_t idesc_s = ptx::umma_idesc_bf16(kKeys, p.head_cols), idesc_o = ptx::umma_idesc_bf16(128, p.head_cols, true, true);
      const uint32_t qa = ptx::smem_u32(q_s), pa = ptx::smem_u32(p_s), ra = ptx::smem_u32(ring);
      // descriptors of the ring's first stage, of Q and of P; addresses in them count 16 bytes
      const uint64_t dk = ptx::umma_desc_k_sw128(ra), dq = ptx::umma_desc_k_sw128(qa);
      const uint64_t dv = ptx::umma_desc_mn_sw128(ra, kPageBlock, 1024), dp = ptx::umma_desc_mn_sw128(pa, kBlock, 1024);
      uint32_t phase = 0u;
      int st = 0;
      auto full = [&]() -> bool {
        if (!ptx::mbar_wait(&ctl->full[st], phase, abort_flag, p.wait_cycles)) return false;
        ptx::tc_fence_after();
        return true;
      };
      auto release = [&]() {
        ptx::umma_commit(&ctl->empty[st]);
        if (++st == p.stages) { st = 0; phase ^= 1u; }
      };
      auto scores = [&](int j) -> bool {
        if (!ptx::mbar_wait(&ctl->s_empty, ((uint32_t)j & 1u) ^ 1u, abort_flag, p.wait_cycles)) return false;
        for (int g = 0; g < G; ++g)
          for (int cb = 0; cb < p.nb; ++cb) {
            if (!full()) return false;
            const uint64_t a = dk + (uint32_t)(st * (kBlock / 16)), bq = dq + (uint32_t)(cb * (kCols * 128 / 16) + g * p.head_cols * (128 / 16));
#pragma unroll
            for (int kk = 0; kk < 4; ++kk)
              ptx::umma_bf16(tmem_s + (uint32_t)(g * p.head_cols), a + kk * 2, bq + kk * 2, idesc_s, (cb > 0 || kk > 0) ? 1u : 0u);
            release();
          }
        ptx::umma_commit(&ctl->s_full);
        return true;
      };
      bool ok = ptx::mbar_wait(&ctl->q_full, 0u, abort_flag, p.wait_cycles);
      if (ok) ok = scores(0);
      for (int j = 0; j < n && ok; ++j) {
        if (j + 1 < n && !scores(j + 1)) break;
        if (!ptx::mbar_wait(&ctl->p_full, (uint32_t)j & 1u, abort_flag, p.wait_cycles)) break;
        for (int i = 0; i < G * 2 && ok; ++i) {
          if (!full()) { ok = false; break; }
          const int col = (i >> 1) * p.head_cols, page = i & 1;
          const uint64_t a = dv + (uint32_t)(st * (kBlock / 16)),
                         bp = dp + (uint32_t)(((col >> 6) * kBlock + (col & 63) * 2 + page * kPageBlock) / 16);
#pragma unroll
          for (int ks = 0; ks < kPageTokens / 16; ++ks)   // 16 keys are 16 rows of 128 bytes further in both tiles
            ptx::umma_bf16(tmem_o + (uint32_t)col, a + ks * 128, bp + ks * 128, idesc_o, (j > 0 || page > 0 || ks > 0) ? 1u : 0u);
          release();
        }
        if (ok) ptx::umma_commit(&ctl->o_done);
      }
    }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 232;");
    // ------------------------------------------------------------------ mixing, softmax, output
    const int quarter = warp & 3, half = warp >> 2, key = quarter * 32 + lane;
    const uint32_t t_lane = (uint32_t)(quarter * 32) << 16;
    const int g8 = lane >> 2, t4 = lane & 3;
    m_s[threadIdx.x] = 0.f;
    softmax_sync();
    float sums[4][4];   // of four groups of 8 columns, the same in every row of the fragment
#pragma unroll
    for (int i = 0; i < 4; ++i) { sums[i][0] = sums[i][1] = sums[i][2] = sums[i][3] = 0.f; }
    // Chunk c of tile j: raw scores of TC tokens and all heads -> mixed scores less their reference points
    auto mix = [&](int j, int c, float2 (&d)[HP][TC / 2]) {
      const int i0 = half * (MT / 2) + c * TC;   // first token
      float2 x[HP][TC / 2];                      // raw scores of the token pairs
#pragma unroll
      for (int h = 0; h < HP; ++h) {
        uint32_t r[TC];
        if (h < H) {   // uniform
          ptx::tmem_ld_32xn<TC>(tmem_s + t_lane + (uint32_t)(p.column[h] + i0), r);
        } else {
#pragma unroll
          for (int i = 0; i < TC; ++i) r[i] = 0u;
        }
#pragma unroll
        for (int i = 0; i < TC / 2; ++i) x[h][i] = make_float2(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1]));
      }
      ptx::tmem_wait_ld();
#pragma unroll
      for (int h = 0; h < HP; ++h) {
        const float* m = m_s + p.column[h] + i0;   // (column 0 for heads that are not there)
        if constexpr (TC >= 4) {
#pragma unroll
          for (int i = 0; i < TC / 4; ++i) {
            const float4 v = *reinterpret_cast<const float4*>(m + 4 * i);
            d[h][2 * i] = make_float2(v.x, v.y);
            d[h][2 * i + 1] = make_float2(v.z, v.w);
          }
        } else {
          d[h][0] = *reinterpret_cast<const float2*>(m);
        }
#pragma unroll
        for (int g = 0; g < HP; ++g)
#pragma unroll
          for (int i = 0; i < TC / 2; ++i) d[h][i] = fma2(talk.t[h * HP + g], x[g][i], d[h][i]);
      }
      if (j * kKeys + kKeys - 1 > base + t0) {   // a tile that the diagonal cuts
        const int first = j * kKeys + key - (base + t0 + i0);   // token i sees this key from i = first on
#pragma unroll
        for (int h = 0; h < HP; ++h)
#pragma unroll
          for (int i = 0; i < TC / 2; ++i) {
            if (first > 2 * i) d[h][i].x = -INFINITY;
            if (first > 2 * i + 1) d[h][i].y = -INFINITY;
          }
      }
    };
    // The chunk's weights into P
    auto weights = [&](int c, const float2 (&d)[HP][TC / 2]) {
#pragma unroll
      for (int h = 0; h < HP; ++h) {
        if (h < H) {
          const int col = p.column[h] + half * (MT / 2) + c * TC;
          uint32_t w[TC / 2];
#pragma unroll
          for (int i = 0; i < TC / 2; ++i) {
            const __nv_bfloat162 v = __floats2bfloat162_rn(ex2_fast(d[h][i].x), ex2_fast(d[h][i].y));
            w[i] = *reinterpret_cast<const uint32_t*>(&v);
          }
          uint8_t* dst = p_s + (col >> 6) * kBlock + key * 128 + ((((col & 63) >> 3) ^ (key & 7)) << 4) + (col & 7) * 2;
          if constexpr (TC == 8) *reinterpret_cast<uint4*>(dst) = make_uint4(w[0], w[1], w[2], w[3]);
          else if constexpr (TC == 4) *reinterpret_cast<uint2*>(dst) = make_uint2(w[0], w[1]);
          else *reinterpret_cast<uint32_t*>(dst) = w[0];
        }
      }
    };
    for (int j = 0; j < (layout_ok ? n : 0); ++j) {
      ptx::mbar_wait(&ctl->s_full, (uint32_t)j & 1u, abort_flag, p.wait_cycles);
      __syncwarp();
      ptx::tc_fence_after();
      volatile uint32_t* grow = &ctl->grow[C::kHalves ? half : 0][j & 1];   // (a fast warp may already be in the next tile)
      bool kept = j == 0;   // this warp has not given the raw scores back
      float2 d[HP][TC / 2];
      if (j > 0) {
#pragma unroll 1
        for (int c = 0; c < 2; ++c) {
          mix(j, c, d);
          float top = -INFINITY;
#pragma unroll
          for (int h = 0; h < HP; ++h)
            if (h < H) {
#pragma unroll
              for (int i = 0; i < TC / 2; ++i) top = max3(top, d[h][i].x, d[h][i].y);
            }
          kept |= __any_sync(0xffffffffu, top > 1.0f) != 0;
          if (c == 0) {   // P of the tile before has been read, by the product and by this half's sums
            half_sync<C::kHalves>(half);
            ptx::mbar_wait(&ctl->o_done, (uint32_t)(j - 1) & 1u, abort_flag, p.wait_cycles);
            __syncwarp();
          } else if (kept) {
            if (lane == 0) *grow = 1u;
          } else {   // the next tile's scores may come, once every warp has said so
            ptx::tc_fence_before();
            __syncwarp();
            if (lane == 0) ptx::mbar_arrive(&ctl->s_empty);
          }
          weights(c, d);
        }
        ptx::fence_proxy_async();   // the weights become visible to the tensor core's reads
      }
      half_sync<C::kHalves>(half);
      const bool again = j == 0 || *grow != 0u;
      if (again) {
        // Uniform over the half's four warps, and rare but for the first tile: the raw scores are still there, since at least
        // one warp has kept them.  New reference points, 2^6 above the maximum, for columns that have outgrown theirs; sums and O
        // follow; the tile's weights once more.
        constexpr int kLowest = (int)0x807fffff;   // -inf in an order of integers that is the order of floats
        int* best = reinterpret_cast<int*>(shift_s);
        const int mine = C::own_column(threadIdx.x);
        ptx::tc_fence_after();
        best[mine] = kLowest;
        half_sync<C::kHalves>(half);
        if ((threadIdx.x & (C::kHalves ? 127 : 255)) == 0) *grow = 0u;
#pragma unroll 1
        for (int c = 0; c < 2; ++c) {
          mix(j, c, d);
#pragma unroll
          for (int h = 0; h < HP; ++h) {
            if (h >= H) continue;
#pragma unroll
            for (int i = 0; i < TC; ++i) {
              const int o = __float_as_int(warp_max((i & 1) ? d[h][i / 2].y : d[h][i / 2].x));
              if (lane == 0) atomicMax(best + p.column[h] + half * (MT / 2) + c * TC + i, o >= 0 ? o : o ^ 0x7fffffff);
            }
          }
        }
        half_sync<C::kHalves>(half);
        {
          const int o = best[mine];
          const float up = __int_as_float(o >= 0 ? o : o ^ 0x7fffffff);
          const float shift = o > kLowest && (j == 0 || up > 0.9f) ? up + 6.0f : 0.f;
          m_s[mine] -= shift;
          shift_s[mine] = shift;
        }
        half_sync<C::kHalves>(half);
        if (j > 0) {   // (the product of the tile before has been waited for above)
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float* by = shift_s + C::eighth(warp, i) * 8 + 2 * t4;
            const float c0 = ex2_fast(-by[0]), c1 = ex2_fast(-by[1]);
            sums[i][0] *= c0; sums[i][1] *= c1; sums[i][2] *= c0; sums[i][3] *= c1;
          }
          for (int v = 0; v < 2 * H; ++v) {
            const int col = p.column[v >> 1] + half * (MT / 2) + (v & 1) * TC;
            uint32_t r[TC];
            ptx::tmem_ld_32xn<TC>(tmem_o + t_lane + (uint32_t)col, r);
            ptx::tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < TC; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * ex2_fast(-shift_s[col + i]));
            ptx::tmem_st_32xn<TC>(tmem_o + t_lane + (uint32_t)col, r);
          }
          ptx::tmem_wait_st();
        }
#pragma unroll 1
        for (int c = 0; c < 2; ++c) {
          mix(j, c, d);
          weights(c, d);
        }
        ptx::tc_fence_before();
        ptx::fence_proxy_async();
        half_sync<C::kHalves>(half);   // every warp has read the raw scores for the last time
        if (kept && lane == 0) ptx::mbar_arrive(&ctl->s_empty);
      }
      if (lane == 0) ptx::mbar_arrive(&ctl->p_full);
      // sums over the keys: ones . P
      const uint32_t ones[4] = {0x3f803f80u, 0x3f803f80u, 0x3f803f80u, 0x3f803f80u};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int col = C::eighth(warp, i) * 8;
        const uint32_t src = s_u32(p_s + (col >> 6) * kBlock);
#pragma unroll
        for (int k = 0; k < kKeys / 32; ++k) {
          uint32_t bb[4];
          const int row = k * 32 + lane;
          ldsm_x4_t(bb, src + (uint32_t)(row * 128 + ((((col & 63) >> 3) ^ (row & 7)) << 4)));
          mma16816(sums[i], ones, bb[0], bb[1]);
          mma16816(sums[i], ones, bb[2], bb[3]);
        }
      }
    }
    // ------------------------------------------------------------------ output
    if (layout_ok) {
      ptx::mbar_wait(&ctl->o_done, (uint32_t)(n - 1) & 1u, abort_flag, p.wait_cycles);
      __syncwarp();
      ptx::tc_fence_after();
      softmax_sync();
      if (g8 == 0) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          float* l = shift_s + C::eighth(warp, i) * 8 + 2 * t4;
          l[0] = sums[i][0];
          l[1] = sums[i][1];
        }
      }
      softmax_sync();
      for (int v = threadIdx.x; v < H * MT; v += kSoftmax) {
        const int h = v / MT, col = p.column[h] + v % MT;
        const float l = shift_s[col] + (p.sink ? ex2_fast(fmaf(__bfloat162float(p.sink[h]), kLog2e, m_s[col])) : 0.f);
        shift_s[col] = 1.0f / l;
      }
      softmax_sync();
      const int dim = quarter * 32 + lane;
      if (!*abort_flag && quarter * 32 < p.value_dim) {
        for (int h = 0; h < H; ++h) {
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            const int i0 = half * (MT / 2) + c * TC, col = p.column[h] + i0;
            uint32_t r[TC];
            ptx::tmem_ld_32xn<TC>(tmem_o + t_lane + (uint32_t)col, r);
            ptx::tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < TC; ++i) {
              const int token = t0 + i0 + i;
              if (token < p.s_new && dim < p.value_dim)
                p.out[((size_t)b * p.s_new + token) * p.out_ld + (size_t)h * p.value_dim + dim] = __float2bfloat16_rn(__uint_as_float(r[i]) * shift_s[col + i]);
            }
          }
        }
      }
    }
  }

  // ------------------------------------------------------------------ teardown
  ptx::tc_fence_before();
  __syncthreads();
  if (*abort_flag && threadIdx.x == 0) {
    p.status[0] = (uint32_t)(-RB_ERR_TIMEOUT); p.status[1] = 0xA711u; p.status[2] = blockIdx.x; p.status[3] = blockIdx.y;
    volatile uint32_t never = 0;   // copies already on their way get a bounded chance to land
    ptx::mbar_wait(&ctl->q_full, 0u, &never, p.wait_cycles);
    const uint32_t issued = ctl->issued;
    for (uint32_t u = issued > (uint32_t)p.stages ? issued - p.stages : 0; u < issued; ++u)
      ptx::mbar_wait(&ctl->full[u % p.stages], (u / p.stages) & 1u, &never, p.wait_cycles);
  }
  __syncthreads();
  if (warp == 9) {
    __syncwarp();
    ptx::tc_fence_after();
    ptx::tmem_dealloc(tmem_s, 512);
  }
}

// columns a key/value head takes: whole 16s that do not cross a block of 64
int head_columns(int n) {
  if (n > 64) return (n + 63) / 64 * 64;
  return n <= 16 ? 16 : n <= 32 ? 32 : 64;
}
int padded_heads(int H) { return H <= 8 ? 8 : H <= 16 ? 16 : 32; }

template <int HP>
int launch_mix(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, MixParams p, const float* talk, float scale) {
  using C = MixShape<HP>;
  constexpr size_t kLimit = 227 * 1024;
  const size_t fixed = C::fixed_bytes(p.nb);
  p.stages = (int)std::min<size_t>(kMaxStages, (kLimit - fixed) / kBlock);
  const size_t smem = fixed + (size_t)p.stages * kBlock;
  MixTalk<HP> coef;
  for (int i = 0; i < HP * HP; ++i) {
    const int h = i / HP, g = i % HP;
    coef.t[i].x = coef.t[i].y = h < p.q_heads && g < p.q_heads ? talk[h * p.q_heads + g] * scale * kLog2e : 0.f;
  }
  auto kern = attention_mix_tc_kernel<HP>;
  static size_t set[64] = {};
  const int dv = ctx->device & 63;
  if (smem > set[dv]) { RB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); set[dv] = smem; }
  CUtensorMap tq, tk, tv;
  const size_t off = (size_t)layer * c->layer_stride_elems();
  const int64_t rows = (int64_t)c->num_pages * c->kv_heads * kPageTokens;
  // q rows are (sequence, position), columns (head, lane): a box is one head's tokens x 64
  RB_TRY(tmap_2d_bf16(ctx, q, (int64_t)batch * p.s_new, (int64_t)p.q_heads * p.D, (int64_t)p.q_heads * p.D, C::MT, &tq));
  RB_TRY(tmap_2d_bf16(ctx, (const bf16*)c->k + off, rows, p.D, p.D, kPageTokens, &tk));
  RB_TRY(tmap_2d_bf16(ctx, (const bf16*)c->v + off, rows, p.D, p.D, kPageTokens, &tv));
  RB_CUDA(launch_kernel(kern, dim3((unsigned)((p.s_new + C::MT - 1) / C::MT), (unsigned)batch), dim3(kThreads), smem, ctx->stream, ctx->pdl, tq, tk,
                        tv, p, coef));
  ctx->launches++;
  return RB_OK;
}

}  // namespace

bool attention_mix_tc_takes(const rb_kv_cache* c, int s_new, int q_heads, const void* q, const AttnExtra& x) {
  if (c->dtype != RB_BF16 || c->shared() || (c->head_dim != 64 && c->head_dim != 128) || q_heads > 32 || q_heads % c->kv_heads != 0) return false;
  if (!x.talk_host || x.window > 0 || x.chunk > 0 || (reinterpret_cast<uintptr_t>(q) & 15) != 0) return false;
  const int mt = kCols / padded_heads(q_heads);
  return s_new >= 16 && c->kv_heads * head_columns(q_heads / c->kv_heads * mt) <= kCols;
}

int attention_mix_tc(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads, float scale, void* out,
                     const AttnExtra& x) {
  MixParams p{};
  const int hp = padded_heads(q_heads);
  p.block_table = c->block_table; p.seq_lens = c->seq_lens; p.pages_per_seq = c->pages_per_seq; p.s_new = s_new; p.q_heads = q_heads;
  p.kv_heads = c->kv_heads; p.group = q_heads / c->kv_heads; p.D = c->head_dim; p.nb = c->head_dim / 64; p.nbv = (x.value_dim + 63) / 64;
  const int mt = kCols / hp;
  p.head_cols = head_columns(p.group * mt);
  for (int h = 0; h < q_heads; ++h) p.column[h] = h / p.group * p.head_cols + h % p.group * mt;
  p.value_dim = x.value_dim;
  p.sink = (const bf16*)x.sink; p.out = (bf16*)out; p.out_ld = x.out_ld; p.status = ctx->status_dev;
  p.wait_cycles = ctx->local_wait_cycles();
  RB_REQUIRE(batch <= 65535, "attention: batch %d too large", batch);
  if (hp == 8) return launch_mix<8>(ctx, q, c, layer, batch, p, x.talk_host, scale);
  if (hp == 16) return launch_mix<16>(ctx, q, c, layer, batch, p, x.talk_host, scale);
  return launch_mix<32>(ctx, q, c, layer, batch, p, x.talk_host, scale);
}

}  // namespace rb
