// What latent attention needs around its attention kernels: the norms of the query's and the cached latent with rotation and cache
// append, the per-head products into the latent's space and out of it, and the head split of prompts whose latents are
// multiplied out.  Single-token calls sum a projection's split-K slabs here.  All arithmetic is float32 but for the tensor-core
// products of the bf16 model.
#include <math.h>

#include <algorithm>
#include <vector>

#include "ctx.h"
#include "mma.cuh"

namespace rb {

namespace {

using bf16 = __nv_bfloat16;

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
int round8(int v) { return (v + 7) / 8 * 8; }

struct Rotation {
  const float *cos_t, *sin_t;   // [position][half]
  int half;                     // pairs that turn
  int interleaved;
};

// Element i of a vector that turns, x(j) giving its elements
template <typename X>
__device__ __forceinline__ float turned(const Rotation& r, int pos, int i, X x) {
  if (i >= 2 * r.half) return x(i);
  const int f = r.interleaved ? i >> 1 : i < r.half ? i : i - r.half;
  const bool first = r.interleaved ? (i & 1) == 0 : i < r.half;
  const float c = r.cos_t[(size_t)pos * r.half + f], s = r.sin_t[(size_t)pos * r.half + f];
  const int j = r.interleaved ? i ^ 1 : first ? i + r.half : i - r.half;
  const float u = x(i), v = x(j);
  return first ? fmaf(u, c, -(v * s)) : fmaf(u, c, v * s);
}

struct Pages {
  const int32_t *block_table, *seq_lens;
  int pages_per_seq, max_seq, kv_heads, D;
};
// where the token of row m sits (s_new rows per sequence); -1: outside the cache
__device__ __forceinline__ int position_of(const Pages& p, int m, int s_new, uint32_t* status) {
  const int pos = p.seq_lens[m / s_new] - s_new + m % s_new;
  if (pos >= 0 && pos < p.max_seq) return pos;
  if (threadIdx.x == 0) { status[0] = (uint32_t)(-RB_ERR_INVALID); status[1] = 0x1A7Eu; status[2] = (uint32_t)pos; }
  return -1;
}
__device__ __forceinline__ size_t page_row(const Pages& p, int m, int s_new, int pos, int head) {
  const int page = p.block_table[(size_t)(m / s_new) * p.pages_per_seq + pos / kPageTokens];
  return (((size_t)page * p.kv_heads + head) * kPageTokens + pos % kPageTokens) * p.D;
}

// ------------------------------------------------------------------------------------------
// Norms, rotation, append.  One block per row; the latent and the key part are staged in shared memory.
// ------------------------------------------------------------------------------------------
template <typename T>
struct AppendArgs {
  const T* src;
  const float* acc;
  int n_acc;
  size_t acc_stride;
  int64_t ld;
  int q_rank, kv_rank, rot_dim, qp, kp, gate, gp;   // padded widths; gate columns
  const T *qw, *kw;
  float eps;
  Rotation rot;
  int s_new, rows;
  Pages pages;
  T *cache, *cq, *latent, *gate_out;
  uint32_t* status;
};

template <typename T, bool kSlabs>
__global__ void __launch_bounds__(256) latent_append_kernel(const AppendArgs<T> a) {
  extern __shared__ float kv_s[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int m = blockIdx.x;
  auto load_u = [&](int col, float* u) {
    if constexpr (!kSlabs) {
      load8(a.src + (size_t)m * a.ld + col, u);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) u[i] = 0.f;
      add_slabs<4>(a.acc, a.n_acc, a.acc_stride, (size_t)m * a.ld + col, u);
    }
  };
  const int pos = position_of(a.pages, m, a.s_new, a.status);
  if (pos < 0) return;   // block-uniform
  // the latent and the key part, and the sum of the latent's squares
  float sk = 0.f, sq = 0.f;
  for (int c = threadIdx.x * 8; c < a.kp; c += blockDim.x * 8) {
    float u[8];
    load_u(a.qp + c, u);
    store8(kv_s + c, u);
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (c + i < a.kv_rank) sk = fmaf(u[i], u[i], sk);
  }
  float q[2][8];   // pieces of the query latent kept in registers; further ones are loaded again
  int n = 0;
  for (int c = threadIdx.x * 8; c < a.qp; c += blockDim.x * 8, ++n) {
    float u[8];
    load_u(c, u);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      sq = fmaf(u[i], u[i], sq);
      if (n == 0) q[0][i] = u[i];
      if (n == 1) q[1][i] = u[i];
    }
  }
  for (int c = threadIdx.x * 8; c < a.gp; c += blockDim.x * 8) {
    float u[8];
    load_u(a.qp + a.kp + c, u);
    store8(a.gate_out + (size_t)m * a.gp + c, u);
  }
  sq = block_sum(sq, red);
  const float rq = 1.0f / sqrtf(sq / (float)a.q_rank + a.eps);
  n = 0;
  for (int c = threadIdx.x * 8; c < a.qp; c += blockDim.x * 8, ++n) {
    float u[8], w[8];
    if (n > 1) load_u(c, u);
    load8(a.qw + c, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) w[i] *= rq * (n == 0 ? q[0][i] : n == 1 ? q[1][i] : u[i]);
    store8(a.cq + (size_t)m * a.qp + c, w);
  }
  if (a.kv_rank == 0) return;
  sk = block_sum(sk, red);   // (its barriers also publish kv_s)
  const float rk = 1.0f / sqrtf(sk / (float)a.kv_rank + a.eps);
  T* row = a.cache + page_row(a.pages, m, a.s_new, pos, 0);
  const int lp = (a.kv_rank + 7) & ~7;
  for (int c = threadIdx.x * 8; c < a.pages.D; c += blockDim.x * 8) {
    float y[8], w[8], z[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = z[i] = 0.f;
    if (c < a.kv_rank) load8(a.kw + c, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int e = c + i;
      if (e < a.kv_rank) y[i] = z[i] = kv_s[e] * rk * w[i];
      else if (e < a.kv_rank + a.rot_dim) y[i] = turned(a.rot, pos, e - a.kv_rank, [&](int j) { return kv_s[a.kv_rank + j]; });
    }
    store8(row + c, y);
    if (a.latent && c < lp) store8(a.latent + (size_t)m * lp + c, z);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const T* __restrict__ cache, const Pages p, int kv_rank, int lp, int s_new,
                                                            int64_t pieces, T* __restrict__ out, uint32_t* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = lp / 8;
  for (int64_t it = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; it < pieces; it += (int64_t)gridDim.x * blockDim.x) {
    const int m = (int)(it / per), c = (int)(it % per) * 8;
    const int pos = position_of(p, m, s_new, status);
    if (pos < 0) continue;
    float v[8];
    load8(cache + page_row(p, m, s_new, pos, 0) + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (c + i >= kv_rank) v[i] = 0.f;
    store8(out + (size_t)m * lp + c, v);
  }
}

// ------------------------------------------------------------------------------------------
// Per-head products: y[row, h, :] = A[row, h, :] . B_h.  Into the latent's space B is [k][n] (rows of uk), out of it [n][k] (rows of
// uv).  bf16: a block has 64 rows x 32 columns of one head, all of K staged at once (a few hundred to a thousand numbers), each
// of four warps 16 rows.  Otherwise one thread per output.
// ------------------------------------------------------------------------------------------
template <typename T>
struct HeadProduct {
  const T* a;                // QUERY: u (bf16 rows), or slabs; else x
  const float* acc;
  int n_acc;
  size_t acc_stride;
  int64_t a_ld;              // row pitch
  int a_head;                // head pitch
  const T* b;
  int64_t b_ld;              // row pitch of the weights
  int heads, n, k;           // columns of the result and length of the product, per head
  int64_t rows;
  T* out;
  int64_t out_ld;
  int out_head;
  // into the latent's space: the turned part behind the product, then zeros up to out_head
  int rot_dim;
  Rotation rot;
  int s_new;
  Pages pages;
  // out of it: the gate
  const T* gate;
  int64_t gate_ld;
  int head_gate;
  uint32_t* status;
};

// what lies behind the product in a query's row, for rows m0 .. m0 + n_rows of head h
// `part` of `parts`: rows are shared out over the blocks that hold the same rows' columns.
template <typename T>
__device__ __forceinline__ void query_tail(const HeadProduct<T>& p, int64_t m0, int n_rows, int h, int part, int parts) {
  const int tail = p.out_head - p.n;
  const int mine = (n_rows - part + parts - 1) / parts;
#pragma unroll 4
  for (int it = threadIdx.x; it < mine * tail; it += blockDim.x) {
    const int r = it / tail, i = it - r * tail;
    const int64_t m = m0 + part + (int64_t)r * parts;
    if (m >= p.rows) continue;
    float y = 0.f;
    if (i < p.rot_dim) {
      const int seq = p.s_new == 1 ? (int)m : (int)(m / p.s_new);
      const int pos = p.pages.seq_lens[seq] - p.s_new + (int)(m - (int64_t)seq * p.s_new);
      if (pos < 0 || pos >= p.pages.max_seq) continue;   // (the append has recorded it)
      const size_t base = (size_t)m * p.a_ld + (size_t)h * p.a_head + p.k;
      y = turned(p.rot, pos, i, [&](int j) {
        if (p.a) return Cvt<T>::to_f(p.a[base + j]);
        float s = 0.f;
        for (int t0 = 0; t0 < p.n_acc; t0 += 4) {
          float v[4];
#pragma unroll
          for (int t = 0; t < 4; ++t) v[t] = t0 + t < p.n_acc ? p.acc[(size_t)(t0 + t) * p.acc_stride + base + j] : 0.f;
#pragma unroll
          for (int t = 0; t < 4; ++t) s += v[t];
        }
        return s;
      });
    }
    p.out[(size_t)m * p.out_ld + (size_t)h * p.out_head + p.n + i] = Cvt<T>::from_f(y);
  }
}

template <typename T>
__device__ __forceinline__ float gate_of(const HeadProduct<T>& p, int64_t m, int h, int c) {
  return p.gate ? sigmoid_f(Cvt<T>::to_f(p.gate[(size_t)m * p.gate_ld + (p.head_gate ? h : h * p.n + c)])) : 1.0f;
}

template <typename T, bool QUERY>
__global__ void __launch_bounds__(128) head_product_plain_kernel(const HeadProduct<T> p) {
  const int64_t m = blockIdx.x;
  const int h = blockIdx.y;
  for (int c = threadIdx.x; c < p.n; c += blockDim.x) {
    float s = 0.f;
    for (int i = 0; i < p.k; ++i) {
      const size_t at = (size_t)m * p.a_ld + (size_t)h * p.a_head + i;
      float x = 0.f;
      if (p.a) x = Cvt<T>::to_f(p.a[at]);
      else
        for (int t = 0; t < p.n_acc; ++t) x += p.acc[(size_t)t * p.acc_stride + at];
      s = fmaf(x, Cvt<T>::to_f(QUERY ? p.b[((size_t)h * p.k + i) * p.b_ld + c] : p.b[((size_t)h * p.n + c) * p.b_ld + i]), s);
    }
    if (!QUERY) s *= gate_of(p, m, h, c);
    p.out[(size_t)m * p.out_ld + (size_t)h * p.out_head + c] = Cvt<T>::from_f(s);
  }
  if (QUERY) query_tail(p, m, 1, h, 0, 1);
}

constexpr int kHpRows = 64, kHpCols = 32, kHpMaxK = 512;

template <bool QUERY>
__global__ void __launch_bounds__(128) head_product_mma_kernel(const HeadProduct<bf16> p, int kc, int vec) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int ap = kc + 8, bp = QUERY ? kHpCols + 8 : kc + 8;   // row pitches
  bf16* a_s = reinterpret_cast<bf16*>(smem);
  bf16* b_s = a_s + kHpRows * ap;
  const int n0 = blockIdx.x * kHpCols, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t m0 = (int64_t)blockIdx.z * kHpRows;
  float o[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  pdl_launch_dependents();
  for (int k0 = 0; k0 < p.k; k0 += kc) {
    const int have = min(kc, p.k - k0);   // zeros from there on
    if (k0 > 0) __syncthreads();
    // weights do not depend on the kernel before this one
    if (QUERY) {   // rows of K, 32 columns; the matrix's rows are padded to a multiple of 8 columns
      for (int it = threadIdx.x; it < kc * (kHpCols / 8); it += blockDim.x) {
        const int r = it / (kHpCols / 8), c = it % (kHpCols / 8) * 8;
        bf16* dst = b_s + r * bp + c;
        if (r < have && n0 + c < p.b_ld) cp_async16(dst, p.b + ((size_t)h * p.k + k0 + r) * p.b_ld + n0 + c);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
      }
    } else {
      for (int it = threadIdx.x; it < kHpCols * (kc / 8); it += blockDim.x) {
        const int r = it / (kc / 8), c = it % (kc / 8) * 8;
        bf16* dst = b_s + r * bp + c;
        if (n0 + r < p.n && k0 + c < p.b_ld) cp_async16(dst, p.b + ((size_t)h * p.n + n0 + r) * p.b_ld + k0 + c);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
      }
    }
    if (k0 == 0) pdl_wait();
    for (int it = threadIdx.x; it < kHpRows * (kc / 8); it += blockDim.x) {
      const int r = it / (kc / 8), c = it % (kc / 8) * 8;
      bf16* dst = a_s + r * ap + c;
      const size_t at = (size_t)(m0 + r) * p.a_ld + (size_t)h * p.a_head + k0 + c;
      if (m0 + r >= p.rows || c >= have) *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
      else if (vec && p.a) cp_async16(dst, p.a + at);
      else if (vec) {
        float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        add_slabs<4>(p.acc, p.n_acc, p.acc_stride, at, v);
        store8(dst, v);
      } else {
        for (int i = 0; i < 8; ++i) {
          float x = 0.f;
          if (c + i < have) {
            if (p.a) x = __bfloat162float(p.a[at + i]);
            else
              for (int t = 0; t < p.n_acc; ++t) x += p.acc[(size_t)t * p.acc_stride + at + i];
          }
          dst[i] = __float2bfloat16_rn(x);
        }
      }
    }
    cp_async_commit();
    if (QUERY && k0 == 0) query_tail(p, m0, kHpRows, h, (int)blockIdx.x, (int)gridDim.x);   // (while the copies land)
    cp_async_wait<0>();
    __syncthreads();
    for (int kk = 0; kk < kc; kk += 16) {
      uint32_t a[4], b0[4], b1[4];
      ldsm_x4(a, s_u32(a_s + (warp * 16 + (lane & 15)) * ap + kk + (lane >> 4) * 8));
      if (QUERY) {   // [k][n]: transposed blocks
        const int r = kk + (lane & 7) + (((lane >> 3) & 1) << 3), c = (lane >> 4) << 3;
        ldsm_x4_t(b0, s_u32(b_s + r * bp + c));
        ldsm_x4_t(b1, s_u32(b_s + r * bp + 16 + c));
      } else {
        const int r = (lane & 7) + ((lane >> 4) << 3), c = kk + (((lane >> 3) & 1) << 3);
        ldsm_x4(b0, s_u32(b_s + r * bp + c));
        ldsm_x4(b1, s_u32(b_s + (16 + r) * bp + c));
      }
      mma16816(o[0], a, b0[0], b0[1]);
      mma16816(o[1], a, b0[2], b0[3]);
      mma16816(o[2], a, b1[0], b1[1]);
      mma16816(o[3], a, b1[2], b1[3]);
    }
  }
  const int g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int64_t m = m0 + warp * 16 + g + hf * 8;
      const int c = n0 + i * 8 + 2 * t;
      if (m >= p.rows) continue;
      bf16* dst = p.out + (size_t)m * p.out_ld + (size_t)h * p.out_head + c;
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (c + e < p.n) dst[e] = __float2bfloat16_rn(QUERY ? o[i][hf * 2 + e] : o[i][hf * 2 + e] * gate_of(p, m, h, c + e));
    }
}

template <typename T, bool QUERY>
int head_product_run(rb_ctx* ctx, const HeadProduct<T>& p) {
  if constexpr (sizeof(T) == 2) {
    if (!ctx->debug_simple_gemm) {
      const int kc = std::min(kHpMaxK, (p.k + 15) / 16 * 16);
      const int vec = (p.k % 8) == 0 && (p.a_head % 8) == 0 && (p.a_ld % 8) == 0 && aligned16(p.a) && aligned16(p.acc);
      const size_t smem = ((size_t)kHpRows * (kc + 8) + (QUERY ? (size_t)kc * (kHpCols + 8) : (size_t)kHpCols * (kc + 8))) * sizeof(bf16);
      auto kern = head_product_mma_kernel<QUERY>;
      static size_t set[64] = {};
      const int dv = ctx->device & 63;
      if (smem > 48 * 1024 && smem > set[dv]) {
        RB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        set[dv] = smem;
      }
      const dim3 grid((unsigned)((p.n + kHpCols - 1) / kHpCols), (unsigned)p.heads, (unsigned)((p.rows + kHpRows - 1) / kHpRows));
      RB_REQUIRE(grid.z <= 65535, "per-head product: too many rows");
      RB_CUDA(launch_kernel(kern, grid, dim3(128), smem, ctx->stream, ctx->pdl, p, kc, vec));
      ctx->launches++;
      return RB_OK;
    }
  }
  head_product_plain_kernel<T, QUERY><<<dim3((unsigned)p.rows, (unsigned)p.heads), 128, 0, ctx->stream>>>(p);
  ctx->launches++;
  return launch_status("head_product_plain");
}

// ------------------------------------------------------------------------------------------
// Heads of a prompt whose latents were multiplied out.  One thread per 8-column piece of a row's q, k or v heads.
// ------------------------------------------------------------------------------------------
template <typename T>
struct HeadsArgs {
  const T *q, *kv;
  int64_t q_ld, kv_ld;
  int v_col, heads, dim, rot_dim, vdim, kv_rank;
  Rotation rot;
  int s_new;
  int64_t rows;
  Pages pages, prompt;       // the latents'; the multiplied-out keys and values'
  const T* cache;
  T *k_out, *v_out, *q_out;
  uint32_t* status;
};

template <typename T, bool kVec>
__global__ void __launch_bounds__(256) latent_heads_kernel(const HeadsArgs<T> a) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = a.prompt.D / 8, H = a.heads, all = 3 * H * per;
  const int qh = a.dim + a.rot_dim;
  const int64_t m = blockIdx.x;
  const int pos = position_of(a.pages, (int)m, a.s_new, a.status);
  if (pos < 0) return;
  const T* key_part = a.cache + page_row(a.pages, (int)m, a.s_new, pos, 0) + a.kv_rank;
  const size_t to = page_row(a.prompt, (int)m, a.s_new, pos, 0);
  for (int it = threadIdx.x; it < all; it += blockDim.x) {
    const int kind = it / (H * per), h = it / per % H, c = it % per * 8;
    const T* src = kind == 0 ? a.q + m * a.q_ld + (size_t)h * qh : kind == 1 ? a.kv + m * a.kv_ld + (size_t)h * a.dim
                                                                             : a.kv + m * a.kv_ld + a.v_col + (size_t)h * a.vdim;
    const int size = kind == 2 ? a.vdim : qh;
    T* dst = (kind == 0 ? a.q_out + (m * H + h) * a.prompt.D : (kind == 1 ? a.k_out : a.v_out) + to + (size_t)h * kPageTokens * a.prompt.D) + c;
    float y[8];
    auto at = [&](int j) { return Cvt<T>::to_f(src[a.dim + j]); };
    if (kVec) {
      if (c >= size) {
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = 0.f;
      } else if (kind == 2 || c < a.dim) {
        *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src + c);
        if (sizeof(T) == 4) *(reinterpret_cast<uint4*>(dst) + 1) = *(reinterpret_cast<const uint4*>(src + c) + 1);
        continue;
      } else if (kind == 1) {
        load8(key_part + c - a.dim, y);
      } else if (a.rot.interleaved && c - a.dim + 8 <= 2 * a.rot.half) {   // four whole pairs
        const int p0 = (c - a.dim) / 2;
        float u[8], cs[4], sn[4];
        load8(src + c, u);
        *reinterpret_cast<float4*>(cs) = *reinterpret_cast<const float4*>(a.rot.cos_t + (size_t)pos * a.rot.half + p0);
        *reinterpret_cast<float4*>(sn) = *reinterpret_cast<const float4*>(a.rot.sin_t + (size_t)pos * a.rot.half + p0);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          y[2 * i] = fmaf(u[2 * i], cs[i], -(u[2 * i + 1] * sn[i]));
          y[2 * i + 1] = fmaf(u[2 * i + 1], cs[i], u[2 * i] * sn[i]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = turned(a.rot, pos, c - a.dim + i, at);
      }
    } else {
      for (int i = 0; i < 8; ++i) {
        const int e = c + i;
        if (e >= size) y[i] = 0.f;
        else if (kind == 2 || e < a.dim) y[i] = Cvt<T>::to_f(src[e]);
        else if (kind == 1) y[i] = Cvt<T>::to_f(key_part[e - a.dim]);
        else y[i] = turned(a.rot, pos, e - a.dim, at);
      }
    }
    store8(dst, y);
  }
}

Pages pages_of(const rb_kv_cache* c) { return Pages{c->block_table, c->seq_lens, c->pages_per_seq, c->max_seq, c->kv_heads, c->head_dim}; }

int check_latent_cache(const char* who, const rb_kv_cache* c, int layer, int kv_rank, int rot_dim, int dtype) {
  RB_REQUIRE(c->shared() && c->kv_heads == 1 && layer >= 0 && layer < c->layers && dtype == c->dtype && kv_rank + rot_dim <= c->head_dim,
             "%s: the cache does not hold latents of this layer", who);
  return RB_OK;
}

}  // namespace

}  // namespace rb

using namespace rb;

extern "C" int32_t rb_latent_append(rb_ctx* ctx, const void* src, const float* acc, int32_t n_acc, int64_t src_ld, int32_t q_rank,
                                    int32_t kv_rank, int32_t rot_dim, const void* qw, const void* kw, float eps, const float* cos_t,
                                    const float* sin_t, int32_t rot_dims, int32_t interleaved, int32_t batch, int32_t s_new,
                                    rb_kv_cache* c, int32_t layer, void* cq, void* latent, void* gate_out, int32_t gate_size, int32_t dtype) {
  RB_REQUIRE(ctx && c && cq && qw && (src || (acc && n_acc > 0)) && (kv_rank == 0 || kw), "rb_latent_append: null argument");
  RB_REQUIRE(batch > 0 && batch <= c->max_batch && s_new > 0 && (src || s_new == 1), "rb_latent_append: bad batch/seq");
  RB_REQUIRE(q_rank > 0 && kv_rank >= 0 && rot_dim >= 0 && rot_dims >= 0 && rot_dims <= rot_dim && (rot_dims % 2) == 0 &&
                 (rot_dims == 0 || (cos_t && sin_t)), "rb_latent_append: bad sizes");
  if (kv_rank > 0) RB_TRY(check_latent_cache("rb_latent_append", c, layer, kv_rank, rot_dim, dtype));
  RB_REQUIRE(aligned16(src) && aligned16(acc) && aligned16(qw) && aligned16(kw) && aligned16(cq) && aligned16(latent) && aligned16(gate_out) &&
                 (src_ld % 8) == 0, "rb_latent_append: buffers must be 16-byte aligned");
  const int64_t rows = (int64_t)batch * s_new;
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    AppendArgs<T> a{};
    a.src = (const T*)src; a.acc = src ? nullptr : acc; a.n_acc = src ? 0 : n_acc; a.acc_stride = (size_t)rows * src_ld; a.ld = src_ld;
    a.q_rank = q_rank; a.kv_rank = kv_rank; a.rot_dim = rot_dim; a.qp = round8(q_rank); a.kp = kv_rank > 0 ? round8(kv_rank + rot_dim) : 0;
    a.gate = gate_size; a.gp = gate_out ? round8(gate_size) : 0;
    RB_REQUIRE(src_ld >= a.qp + a.kp + a.gp, "rb_latent_append: row pitch %lld does not hold the parts", (long long)src_ld);
    a.qw = (const T*)qw; a.kw = (const T*)kw; a.eps = eps; a.rot = Rotation{cos_t, sin_t, rot_dims / 2, interleaved};
    a.s_new = s_new; a.rows = (int)rows; a.pages = pages_of(c);
    a.cache = kv_rank > 0 ? (T*)c->k + (size_t)layer * c->layer_stride_elems() : nullptr;
    a.cq = (T*)cq; a.latent = (T*)latent; a.gate_out = (T*)gate_out; a.status = ctx->status_dev;
    const double C = a.qp + a.kp, es = sizeof(T);
    ProfScope prof(ctx, RB_PROF_ROPE_KV, (double)rows * ((src ? es * C : 4.0 * n_acc * (C + a.gp) + es * a.gp) + es * C + (latent ? es * kv_rank : 0.0)), 0.0);
    const int threads = std::min(256, std::max(64, (std::max(a.qp, a.kp) / 8 + 31) / 32 * 32));
    const size_t smem = (size_t)a.kp * sizeof(float);
    RB_REQUIRE(smem <= 48 * 1024, "rb_latent_append: a latent of %d is too large", kv_rank);
    RB_CUDA(launch_kernel(src ? latent_append_kernel<T, false> : latent_append_kernel<T, true>, dim3((unsigned)rows), dim3(threads), smem,
                          ctx->stream, ctx->pdl, a));
    ctx->launches++;
    return RB_OK;
  };
  if (dtype == RB_BF16) return fill(bf16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_latent_append: dtype %d unsupported", dtype);
}

extern "C" int32_t rb_latent_gather(rb_ctx* ctx, rb_kv_cache* c, int32_t layer, int32_t kv_rank, int32_t batch, int32_t s_new, void* out,
                                    int32_t dtype) {
  RB_REQUIRE(ctx && c && out && aligned16(out) && kv_rank > 0, "rb_latent_gather: bad argument");
  RB_REQUIRE(batch > 0 && batch <= c->max_batch && s_new > 0, "rb_latent_gather: bad batch/seq");
  RB_TRY(check_latent_cache("rb_latent_gather", c, layer, kv_rank, 0, dtype));
  const int64_t rows = (int64_t)batch * s_new, pieces = rows * (round8(kv_rank) / 8);
  const int blocks = (int)std::min<int64_t>((pieces + 255) / 256, 16 * ctx->sm_count);
  ProfScope prof(ctx, RB_PROF_ROPE_KV, 2.0 * rows * kv_rank * dtype_size(dtype), 0.0);
  auto go = [&](auto tag) -> int {
    using T = decltype(tag);
    RB_CUDA(launch_kernel(latent_gather_kernel<T>, dim3((unsigned)blocks), dim3(256), 0, ctx->stream, ctx->pdl,
                          (const T*)c->k + (size_t)layer * c->layer_stride_elems(), pages_of(c), kv_rank, round8(kv_rank), s_new, pieces,
                          (T*)out, ctx->status_dev));
    ctx->launches++;
    return RB_OK;
  };
  if (dtype == RB_BF16) return go(bf16());
  if (dtype == RB_F32) return go(float());
  return fail(RB_ERR_DTYPE, "rb_latent_gather: dtype %d unsupported", dtype);
}

extern "C" int32_t rb_latent_query(rb_ctx* ctx, const void* src, const float* acc, int32_t n_acc, int64_t src_ld, const void* uk,
                                   int32_t heads, int32_t dim, int32_t rot_dim, int32_t kv_rank, const float* cos_t, const float* sin_t,
                                   int32_t rot_dims, int32_t interleaved, int32_t batch, int32_t s_new, rb_kv_cache* c, void* out,
                                   int32_t dtype) {
  RB_REQUIRE(ctx && c && uk && out && (src || (acc && n_acc > 0)), "rb_latent_query: null argument");
  RB_REQUIRE(batch > 0 && batch <= c->max_batch && s_new > 0, "rb_latent_query: bad batch/seq");
  RB_REQUIRE(heads > 0 && dim > 0 && kv_rank > 0 && rot_dim >= 0 && rot_dims >= 0 && rot_dims <= rot_dim && (rot_dims % 2) == 0 &&
                 src_ld >= (int64_t)heads * (dim + rot_dim) && (rot_dims == 0 || (cos_t && sin_t)), "rb_latent_query: bad sizes");
  RB_TRY(check_latent_cache("rb_latent_query", c, 0, kv_rank, rot_dim, dtype));
  RB_REQUIRE(aligned16(uk) && aligned16(out), "rb_latent_query: buffers must be 16-byte aligned");
  const int64_t rows = (int64_t)batch * s_new;
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    HeadProduct<T> p{};
    p.a = (const T*)src; p.acc = src ? nullptr : acc; p.n_acc = src ? 0 : n_acc; p.acc_stride = (size_t)rows * src_ld; p.a_ld = src_ld;
    p.a_head = dim + rot_dim; p.b = (const T*)uk; p.b_ld = round8(kv_rank); p.heads = heads; p.n = kv_rank; p.k = dim; p.rows = rows;
    p.out = (T*)out; p.out_ld = (int64_t)heads * c->head_dim; p.out_head = c->head_dim; p.rot_dim = rot_dim;
    p.rot = Rotation{cos_t, sin_t, rot_dims / 2, interleaved}; p.s_new = s_new; p.pages = pages_of(c); p.status = ctx->status_dev;
    const double es = sizeof(T);
    ProfScope prof(ctx, RB_PROF_GEMM, es * heads * ((double)dim * kv_rank + (double)rows * (dim + 2.0 * rot_dim + kv_rank)),
                   2.0 * rows * heads * (double)dim * kv_rank);
    return head_product_run<T, true>(ctx, p);
  };
  if (dtype == RB_BF16) return fill(bf16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_latent_query: dtype %d unsupported", dtype);
}

extern "C" int32_t rb_latent_output(rb_ctx* ctx, const void* x, const void* uv, int32_t heads, int32_t kv_rank, int32_t value_dim,
                                    const void* gate, int64_t gate_ld, int32_t head_gate, int64_t rows, void* out, int64_t out_ld,
                                    int32_t dtype) {
  RB_REQUIRE(ctx && x && uv && out, "rb_latent_output: null argument");
  RB_REQUIRE(heads > 0 && kv_rank > 0 && value_dim > 0 && rows >= 0 && out_ld >= (int64_t)heads * value_dim, "rb_latent_output: bad sizes");
  RB_REQUIRE(aligned16(x) && aligned16(uv), "rb_latent_output: buffers must be 16-byte aligned");
  if (rows == 0) return RB_OK;
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    HeadProduct<T> p{};
    const int kp = round8(kv_rank);
    p.a = (const T*)x; p.a_ld = (int64_t)heads * kp; p.a_head = kp; p.b = (const T*)uv; p.b_ld = kp; p.heads = heads; p.n = value_dim; p.k = kp;
    p.rows = rows; p.out = (T*)out; p.out_ld = out_ld; p.out_head = value_dim; p.gate = (const T*)gate; p.gate_ld = gate_ld;
    p.head_gate = head_gate; p.s_new = 1; p.status = ctx->status_dev;
    const double es = sizeof(T);
    ProfScope prof(ctx, RB_PROF_GEMM, es * heads * ((double)value_dim * kv_rank + (double)rows * (value_dim * (gate && !head_gate ? 2.0 : 1.0) + kv_rank)),
                   2.0 * rows * heads * (double)value_dim * kv_rank);
    return head_product_run<T, false>(ctx, p);
  };
  if (dtype == RB_BF16) return fill(bf16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_latent_output: dtype %d unsupported", dtype);
}

extern "C" int32_t rb_latent_heads(rb_ctx* ctx, const void* q, int64_t q_ld, const void* kv, int64_t kv_ld, int32_t v_col, int32_t heads,
                                   int32_t dim, int32_t rot_dim, int32_t value_dim, int32_t kv_rank, const float* cos_t, const float* sin_t,
                                   int32_t rot_dims, int32_t interleaved, int32_t batch, int32_t s_new, rb_kv_cache* c, int32_t layer,
                                   rb_kv_cache* prompt, void* q_out, int32_t dtype) {
  RB_REQUIRE(ctx && q && kv && c && prompt && q_out, "rb_latent_heads: null argument");
  RB_REQUIRE(batch > 0 && batch <= c->max_batch && s_new > 0, "rb_latent_heads: bad batch/seq");
  RB_REQUIRE(heads > 0 && heads == prompt->kv_heads && dtype == prompt->dtype && !prompt->shared() && dim > 0 && value_dim > 0 &&
                 dim + rot_dim <= prompt->head_dim && value_dim <= prompt->head_dim && s_new <= prompt->pages_per_seq * kPageTokens &&
                 batch * prompt->pages_per_seq <= prompt->num_pages, "rb_latent_heads: the prompt's cache does not fit");
  RB_REQUIRE(rot_dims >= 0 && rot_dims <= rot_dim && (rot_dims % 2) == 0 && (rot_dims == 0 || (cos_t && sin_t)), "rb_latent_heads: bad sizes");
  RB_TRY(check_latent_cache("rb_latent_heads", c, layer, kv_rank, rot_dim, dtype));
  for (int b = 0; b < batch; ++b) RB_REQUIRE(c->host_lens[b] == s_new, "rb_latent_heads: sequence %d does not start here", b);
  const int64_t rows = (int64_t)batch * s_new;
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    HeadsArgs<T> a{};
    a.q = (const T*)q; a.kv = (const T*)kv; a.q_ld = q_ld; a.kv_ld = kv_ld; a.v_col = v_col; a.heads = heads; a.dim = dim; a.rot_dim = rot_dim;
    a.vdim = value_dim; a.kv_rank = kv_rank; a.rot = Rotation{cos_t, sin_t, rot_dims / 2, interleaved}; a.s_new = s_new; a.rows = rows;
    a.pages = pages_of(c); a.prompt = pages_of(prompt); a.cache = (const T*)c->k + (size_t)layer * c->layer_stride_elems();
    a.k_out = (T*)prompt->k; a.v_out = (T*)prompt->v; a.q_out = (T*)q_out; a.status = ctx->status_dev;
    const bool vec = (dim % 8) == 0 && (rot_dim % 8) == 0 && (value_dim % 8) == 0 && (kv_rank % 8) == 0 && (v_col % 8) == 0 && (q_ld % 8) == 0 &&
                     (kv_ld % 8) == 0 && (rot_dims % 8) == 0 && aligned16(q) && aligned16(kv) && aligned16(q_out) && aligned16(cos_t) && aligned16(sin_t);
    const double es = sizeof(T), read = heads * (2.0 * dim + rot_dim + value_dim) + rot_dim, wrote = heads * (2.0 * (dim + rot_dim) + value_dim);
    ProfScope prof(ctx, RB_PROF_ROPE_KV, es * rows * (read + wrote), 0.0);
    const int items = 3 * heads * (prompt->head_dim / 8), threads = std::min(256, (items + 31) / 32 * 32);
    RB_CUDA(launch_kernel(vec ? latent_heads_kernel<T, true> : latent_heads_kernel<T, false>, dim3((unsigned)rows), dim3(threads), 0,
                          ctx->stream, ctx->pdl, a));
    ctx->launches++;
    return RB_OK;
  };
  if (dtype == RB_BF16) return fill(bf16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_latent_heads: dtype %d unsupported", dtype);
}
