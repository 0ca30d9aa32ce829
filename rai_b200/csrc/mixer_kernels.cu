// Kernels of the layer-by-layer designs (layered.cu): a float32 residual stream with the norm on a sublayer's output,
// the short causal convolution with query/key norm and cache append, and the HGRN2 recurrence.  Rows have a pitch that
// is a multiple of 8 elements and zero padding, so every row access is a 16-byte piece; all arithmetic is float32.
#include <algorithm>

#include "ctx.h"

namespace rb {

namespace {

// ------------------------------------------------------------------------------------------
// Embedding into the residual stream.  One block per id; `ld` columns (the table has the same pitch).
// ------------------------------------------------------------------------------------------
template <typename T>
__global__ void embed_stream_kernel(const T* __restrict__ table, const uint32_t* __restrict__ ids, int64_t vocab, int ld,
                                    float* __restrict__ h, T* __restrict__ x, uint32_t* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = blockIdx.x;
  uint32_t id = ids[i];
  if (id >= (uint64_t)vocab) {  // record and clamp: never read out of bounds, never trap
    if (threadIdx.x == 0) { status[0] = (uint32_t)(-RB_ERR_INVALID); status[1] = 0xE3BEDu; status[2] = id; }
    id = (uint32_t)(vocab - 1);
  }
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {
    float v[8];
    load8(table + (size_t)id * ld + c, v);
    store8(h + (size_t)i * ld + c, v);
    if (x) store8(x + (size_t)i * ld + c, v);
  }
}

// ------------------------------------------------------------------------------------------
// h += y / rms(y) * gain, x = h in the model dtype; y = tensor and/or split-K slabs.  One block per row (several rows
// per block at prefill sizes); the row stays in registers between the sum of squares and the scaling.
// ------------------------------------------------------------------------------------------
template <typename T, int kChunks, bool kSlabs>
__global__ void __launch_bounds__(512) add_scaled_norm_kernel(const T* __restrict__ y, const float* __restrict__ acc, int n_acc,
                                                              size_t acc_stride, const T* __restrict__ gain, float eps, int width,
                                                              int ld, float* __restrict__ h, T* __restrict__ x, int64_t n_rows) {
  __shared__ float red[32];
  pdl_launch_dependents();
  const float g = Cvt<T>::to_f(gain[0]);
  const int nchunk = ld >> 3;
  pdl_wait();
  for (int64_t row = blockIdx.x; row < n_rows; row += gridDim.x) {
    const size_t base = (size_t)row * ld;
    float v[kChunks][8], hv[kChunks][8];
    float s = 0.f;
#pragma unroll
    for (int c = 0; c < kChunks; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
#pragma unroll
      for (int i = 0; i < 8; ++i) v[c][i] = 0.f;
      if (ch >= nchunk) continue;
      load8(h + base + ch * 8, hv[c]);
      if (y) load8(y + base + ch * 8, v[c]);
      if (kSlabs) add_slabs(acc, n_acc, acc_stride, base + ch * 8, v[c]);
#pragma unroll
      for (int i = 0; i < 8; ++i) s += v[c][i] * v[c][i];
    }
    s = block_sum(s, red);
    const float r = g / sqrtf(s / (float)width + eps);
#pragma unroll
    for (int c = 0; c < kChunks; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch >= nchunk) continue;
#pragma unroll
      for (int i = 0; i < 8; ++i) hv[c][i] = fmaf(v[c][i], r, hv[c][i]);
      store8(h + base + ch * 8, hv[c]);
      if (x) store8(x + base + ch * 8, hv[c]);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(512) scalar_norm_rows_kernel(const float* __restrict__ h, const int32_t* __restrict__ rows,
                                                               int64_t row_step, const T* __restrict__ gain, float eps, int width,
                                                               int ld, T* __restrict__ out) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t src = rows ? rows[blockIdx.x] : (blockIdx.x + 1) * row_step - 1;
  const float* p = h + (size_t)src * ld;
  float s = 0.f;
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {
    float v[8];
    load8(p + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) s += v[i] * v[i];
  }
  s = block_sum(s, red);
  const float r = Cvt<T>::to_f(gain[0]) / sqrtf(s / (float)width + eps);
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {
    float v[8];
    load8(p + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= r;
    store8(out + (size_t)blockIdx.x * ld + c, v);
  }
}

// ------------------------------------------------------------------------------------------
// Convolution over time, query / key norm, head split, cache append.  A block takes `per_block` consecutive rows; each
// thread keeps to its own 8-channel pieces, so the taps of neighbouring rows are found in L1.
// ------------------------------------------------------------------------------------------
template <typename T>
struct ConvArgs {
  const T* src;
  const float* acc;
  int n_acc;
  size_t acc_stride;
  const T *bias, *conv, *qw, *kw;
  int taps, s_new, q_heads, kv_heads, kd, vd, D;
  int qp, kp, vp, gp;          // padded widths of the four parts
  int64_t ld;
  float eps;
  T *kc, *vc;
  const int32_t *block_table, *seq_lens, *slots, *new_lens;
  int pages_per_seq, max_seq, rows, per_block;
  float* ring;
  T *q_out, *gate_out;
  uint32_t* status;
};

template <typename T>
__global__ void __launch_bounds__(256) conv_norm_append_kernel(const ConvArgs<T> a) {
  extern __shared__ float row_s[];  // one row of q, k, v after the convolution
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int C = a.qp + a.kp + a.vp, hist = a.taps - 1;
  const bool vec = (a.kd % 8) == 0 && (a.vd % 8) == 0;
  auto load_u = [&](size_t m, int c, float* u) {  // the projection's row m, columns c..c+8, with its bias
#pragma unroll
    for (int i = 0; i < 8; ++i) u[i] = 0.f;
    float t[8];
    if (a.src) load8(a.src + m * a.ld + c, u);
    add_slabs<4>(a.acc, a.n_acc, a.acc_stride, m * a.ld + c, u);
    if (a.bias && !a.src) { load8(a.bias + c, t);   // a finished tensor already has its bias
#pragma unroll
      for (int i = 0; i < 8; ++i) u[i] += t[i]; }
  };
  for (int m = blockIdx.x * a.per_block; m < min(a.rows, (int)(blockIdx.x + 1) * a.per_block); ++m) {
    const int b = m / a.s_new, s = m % a.s_new;
    const int base = a.seq_lens[b] - a.s_new, pos = base + s;
    if (pos < 0 || pos >= a.max_seq) {  // block-uniform
      if (threadIdx.x == 0) { a.status[0] = (uint32_t)(-RB_ERR_INVALID); a.status[1] = 0xC0ABu; a.status[2] = (uint32_t)pos; }
      continue;
    }
    const bool is_token = !a.new_lens || s < a.new_lens[b];
    float* ring = hist > 0 ? a.ring + (size_t)a.slots[b] * hist * C : nullptr;
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x * 8; c < C; c += blockDim.x * 8) {
      float y[8], u[8], w[8];
      load_u(m, c, u);
      load8(a.conv + (size_t)hist * C + c, w);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] = w[i] * u[i];
      for (int back = 1; back <= hist; ++back) {
        float o[8];
        if (s >= back) load_u(m - back, c, o);
        else if (pos >= back) load8(ring + (size_t)((pos - back) % hist) * C + c, o);
        else break;
        load8(a.conv + (size_t)(hist - back) * C + c, w);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = fmaf(w[i], o[i], y[i]);
      }
      // a single-token step replaces the oldest value, which this thread has just read
      if (a.s_new == 1 && hist > 0 && is_token) store8(ring + (size_t)(pos % hist) * C + c, u);
      float s2 = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) s2 = fmaf(y[i], y[i], s2);
      if (c < a.qp) sq += s2; else if (c < a.qp + a.kp) sk += s2;
      store8(row_s + c, y);
    }
    if (a.gate_out)
      for (int c = threadIdx.x * 8; c < a.gp; c += blockDim.x * 8) {
        float u[8];
        load_u(m, C + c, u);
        store8(a.gate_out + (size_t)m * a.gp + c, u);
      }
    sq = block_sum(sq, red);   // its barriers also publish row_s
    if (a.kv_heads > 0) sk = block_sum(sk, red);
    const float rq = a.qw ? 1.0f / sqrtf(sq / (float)(a.q_heads * a.kd) + a.eps) : 1.0f;
    const float rk = a.kw ? 1.0f / sqrtf(sk / (float)(max(a.kv_heads, 1) * a.kd) + a.eps) : 1.0f;
    const int page = a.kv_heads > 0 ? a.block_table[(size_t)b * a.pages_per_seq + pos / kPageTokens] : 0;
    T* q_row = a.q_out + (size_t)m * a.q_heads * a.D;
    auto kv_row = [&](T* cache, int g) { return cache + (((size_t)page * a.kv_heads + g) * kPageTokens + pos % kPageTokens) * a.D; };
    if (vec) {
      const int dq = a.D / 8, nk = a.kd / 8, nv = a.vd / 8;
      const int items_q = a.q_heads * dq, items_k = a.kv_heads * nk, items_v = a.kv_heads * nv;
      for (int it = threadIdx.x; it < items_q + items_k + items_v; it += blockDim.x) {
        float y[8], w[8];
        if (it < items_q) {
          const int h = it / dq, i0 = (it % dq) * 8;
#pragma unroll
          for (int i = 0; i < 8; ++i) y[i] = 0.f;
          if (i0 < a.kd) {
            load8(row_s + h * a.kd + i0, y);
            if (a.qw) { load8(a.qw + h * a.kd + i0, w);
#pragma unroll
              for (int i = 0; i < 8; ++i) y[i] = y[i] * rq * w[i]; }
          }
          store8(q_row + h * a.D + i0, y);
        } else if (it < items_q + items_k) {
          const int j = it - items_q, g = j / nk, i0 = (j % nk) * 8;
          load8(row_s + a.qp + g * a.kd + i0, y);
          if (a.kw) { load8(a.kw + g * a.kd + i0, w);
#pragma unroll
            for (int i = 0; i < 8; ++i) y[i] = y[i] * rk * w[i]; }
          store8(kv_row(a.kc, g) + i0, y);
        } else {
          const int j = it - items_q - items_k, g = j / nv, i0 = (j % nv) * 8;
          load8(row_s + a.qp + a.kp + g * a.vd + i0, y);
          store8(kv_row(a.vc, g) + i0, y);
        }
      }
    } else {
      for (int it = threadIdx.x; it < a.q_heads * a.D; it += blockDim.x) {
        const int h = it / a.D, i = it % a.D;
        float y = 0.f;
        if (i < a.kd) y = row_s[h * a.kd + i] * (a.qw ? rq * Cvt<T>::to_f(a.qw[h * a.kd + i]) : 1.0f);
        q_row[it] = Cvt<T>::from_f(y);
      }
      for (int it = threadIdx.x; it < a.kv_heads * a.kd; it += blockDim.x)
        kv_row(a.kc, it / a.kd)[it % a.kd] = Cvt<T>::from_f(row_s[a.qp + it] * (a.kw ? rk * Cvt<T>::to_f(a.kw[it]) : 1.0f));
      for (int it = threadIdx.x; it < a.kv_heads * a.vd; it += blockDim.x)
        kv_row(a.vc, it / a.vd)[it % a.vd] = Cvt<T>::from_f(row_s[a.qp + a.kp + it]);
    }
    __syncthreads();  // row_s is rewritten by the next row
  }
}

// The last taps - 1 projected values of every sequence of a multi-token call, once all its rows have been convolved.
template <typename T>
__global__ void conv_ring_save_kernel(const ConvArgs<T> a) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, C = a.qp + a.kp + a.vp, hist = a.taps - 1;
  const int base = a.seq_lens[b] - a.s_new, valid = a.new_lens ? a.new_lens[b] : a.s_new;
  float* ring = a.ring + (size_t)a.slots[b] * hist * C;
  for (int s = max(0, valid - hist); s < valid; ++s)
    for (int c = threadIdx.x * 8; c < C; c += blockDim.x * 8) {
      float u[8];
      load8(a.src + ((size_t)b * a.s_new + s) * a.ld + c, u);
      store8(ring + (size_t)((base + s) % hist) * C + c, u);
    }
}

// ------------------------------------------------------------------------------------------
// HGRN2.  One block owns a whole head's state S [key_dim][value_dim] in registers and walks tokens: a lane holds
// kRows rows x 8 columns (16 row groups x 2 column groups per warp, 16 columns per warp), so a token costs three FMA-pipe
// operations per state element (k v, f S + k v, S q) and o_t needs a reduction over 16 lanes.  Gates, keys and values
// of 16 tokens at a time are prepared in shared memory.
//
// A prompt is cut into pieces that run side by side: pass 1 (OUT = false) runs the recurrence of each piece from zero and
// leaves its final state and the product of its forget gates; hgrn2_carry_kernel turns these into the state in front
// of each piece; pass 2 (OUT = true) runs the recurrence again from there.  No gate is ever divided by, so long
// decays cannot overflow, and the arithmetic of a token does not depend on where the cuts fall.
// ------------------------------------------------------------------------------------------
constexpr int kTileTokens = 16;

template <typename T>
struct HgrnArgs {
  const T* src;
  const float* acc;
  int n_acc;
  size_t acc_stride;
  int64_t ld, out_ld;
  const T *f_bias, *lower, *norm_w;
  float eps;
  int heads, dim, vdim, f_off, v_off;
  int s_new, piece, n_pieces;
  const int32_t *seq_lens, *slots, *new_lens;
  float* state;   // [slot][head][dim][vdim]
  float* carry;   // [batch][head][piece][dim][vdim]
  float* decay;   // [batch][head][piece][dim]
  T* out;
};

template <typename T, int kRows, bool OUT, int kMaxThreads>
__global__ void __launch_bounds__(kMaxThreads) hgrn2_kernel(const HgrnArgs<T> a) {
  constexpr int DP = kRows * 16;
  extern __shared__ __align__(16) float sm[];
  const int n_warps = blockDim.x >> 5, cols = n_warps * 16;
  float* q_s = sm;                          // [tokens][DP]
  float* f_s = q_s + kTileTokens * DP;
  float* k_s = f_s + kTileTokens * DP;
  float* v_s = k_s + kTileTokens * DP;      // [tokens][cols]
  float* o_s = v_s + kTileTokens * cols;    // [tokens][cols]
  float* g_s = o_s + kTileTokens * cols;    // [DP] product of the gates (pass 1)
  const int piece = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rg = lane & 15, c0 = warp * 16 + (lane >> 4) * 8;
  pdl_launch_dependents();
  // A single-token step reads its lengths and state before it waits: both were left by work that a kernel without early
  // release (the one that advances the lengths) separates from this step.
  const bool early = a.s_new == 1;
  if (!early) pdl_wait();
  const int base = __ldcg(a.seq_lens + b) - a.s_new;
  const int valid = a.new_lens ? __ldcg(a.new_lens + b) : a.s_new;
  const int t_lo = piece * a.piece, t_hi = min(t_lo + a.piece, valid);
  const bool last = t_hi == valid;
  if (t_lo >= t_hi || (!OUT && last)) {
    if (early) pdl_wait();
    return;
  }
  const size_t elems = (size_t)a.dim * a.vdim;
  float* slot_state = a.state + ((size_t)a.slots[b] * a.heads + h) * elems;
  const size_t pc = ((size_t)b * a.heads + h) * a.n_pieces + piece;
  float S[kRows][8];
  const float* from = nullptr;
  if (OUT) from = a.n_pieces > 1 ? a.carry + pc * elems : base > 0 ? slot_state : nullptr;
  const bool vec4 = (a.vdim & 3) == 0;
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    const int row = (r >> 2) * 64 + rg * 4 + (r & 3);
#pragma unroll
    for (int c = 0; c < 8; ++c) S[r][c] = 0.f;
    if (from && row < a.dim) {
      const float* p = from + (size_t)row * a.vdim + c0;
#pragma unroll
      for (int c = 0; c < 8; c += 4) {
        if (vec4) {
          if (c0 + c < a.vdim) {
            const float4 t = __ldcg(reinterpret_cast<const float4*>(p + c));
            S[r][c] = t.x; S[r][c + 1] = t.y; S[r][c + 2] = t.z; S[r][c + 3] = t.w;
          }
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (c0 + c + j < a.vdim) S[r][c + j] = __ldcg(p + c + j);
        }
      }
    }
  }
  if (early) pdl_wait();
  if (!OUT)
    for (int i = threadIdx.x; i < DP; i += blockDim.x) g_s[i] = 1.f;

  auto load_u = [&](size_t m, int col) {
    float u = a.src ? Cvt<T>::to_f(a.src[m * a.ld + col]) : 0.f;
    for (int k = 0; k < a.n_acc; ++k) u += a.acc[(size_t)k * a.acc_stride + m * a.ld + col];
    return u;
  };

  for (int t0 = t_lo; t0 < t_hi; t0 += kTileTokens) {
    const int nt = min(kTileTokens, t_hi - t0);
    // ---- gates, keys, queries and values of this tile
    for (int i = threadIdx.x; i < nt * DP; i += blockDim.x) {
      const int t = i / DP, c = i % DP;
      float q = 0.f, f = 0.f, k = 0.f;
      if (c < a.dim) {
        const size_t m = (size_t)b * a.s_new + t0 + t;
        const int ch = h * a.dim + c;
        if (OUT) { const float u = load_u(m, ch); q = u * sigmoid_f(u); }
        const float z = load_u(m, a.f_off + ch) + Cvt<T>::to_f(a.f_bias[ch]);
        const float lo = Cvt<T>::to_f(a.lower[ch]);
        const float e = expf(-z), sg = 1.0f / (1.0f + e);
        f = fmaf(1.0f - lo, sg, lo);
        // 1 - f = (1 - lower) sigmoid(-z), formed without the cancellation of 1 - f
        k = (1.0f - lo) * (z > 0.f ? e * sg : 1.0f - sg);
      }
      if (OUT) q_s[i] = q;
      f_s[i] = f;
      k_s[i] = k;
    }
    for (int i = threadIdx.x; i < nt * cols; i += blockDim.x) {
      const int t = i / cols, c = i % cols;
      v_s[i] = c < a.vdim ? load_u((size_t)b * a.s_new + t0 + t, a.v_off + h * a.vdim + c) : 0.f;
    }
    __syncthreads();
    if (!OUT)
      for (int i = threadIdx.x; i < DP; i += blockDim.x) {
        float g = g_s[i];
        for (int t = 0; t < nt; ++t) g *= f_s[t * DP + i];
        g_s[i] = g;
      }
    // ---- the recurrence
    for (int t = 0; t < nt; ++t) {
      const float4 va = *reinterpret_cast<const float4*>(v_s + t * cols + c0);
      const float4 vb = *reinterpret_cast<const float4*>(v_s + t * cols + c0 + 4);
      const float v[8] = {va.x, va.y, va.z, va.w, vb.x, vb.y, vb.z, vb.w};
      float o[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int r4 = 0; r4 < kRows / 4; ++r4) {
        const int at = t * DP + r4 * 64 + rg * 4;
        const float4 f4 = *reinterpret_cast<const float4*>(f_s + at);
        const float4 k4 = *reinterpret_cast<const float4*>(k_s + at);
        float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f);
        if (OUT) q4 = *reinterpret_cast<const float4*>(q_s + at);
        const float fr[4] = {f4.x, f4.y, f4.z, f4.w}, kr[4] = {k4.x, k4.y, k4.z, k4.w}, qr[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          float* row = S[r4 * 4 + j];
#pragma unroll
          for (int c = 0; c < 8; ++c) {
            row[c] = fmaf(fr[j], row[c], kr[j] * v[c]);
            if (OUT) o[c] = fmaf(row[c], qr[j], o[c]);
          }
        }
      }
      if (OUT) {
        // sum over the 16 row groups; each exchange halves the columns a lane is responsible for
        const bool b3 = lane & 8, b2 = lane & 4, b1 = lane & 2;
        float p4[4], p2[2];
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float got = __shfl_xor_sync(0xffffffffu, b3 ? o[c] : o[c + 4], 8);
          p4[c] = (b3 ? o[c + 4] : o[c]) + got;
        }
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const float got = __shfl_xor_sync(0xffffffffu, b2 ? p4[c] : p4[c + 2], 4);
          p2[c] = (b2 ? p4[c + 2] : p4[c]) + got;
        }
        float p1 = (b1 ? p2[1] : p2[0]) + __shfl_xor_sync(0xffffffffu, b1 ? p2[0] : p2[1], 2);
        p1 += __shfl_xor_sync(0xffffffffu, p1, 1);
        if ((lane & 1) == 0) o_s[t * cols + c0 + (b3 ? 4 : 0) + (b2 ? 2 : 0) + (b1 ? 1 : 0)] = p1;
      }
    }
    __syncthreads();
    if (OUT) {
      // ---- norm over the head's values, one warp per token (the next tile's staging touches other arrays)
      for (int t = warp; t < nt; t += n_warps) {
        float s = 0.f;
        for (int c = lane; c < a.vdim; c += 32) { const float y = o_s[t * cols + c]; s = fmaf(y, y, s); }
        s = warp_sum(s);
        const float r = 1.0f / sqrtf(s / (float)a.vdim + a.eps);
        T* dst = a.out + ((size_t)b * a.s_new + t0 + t) * a.out_ld + (size_t)h * a.vdim;
        for (int c = lane; c < a.vdim; c += 32) dst[c] = Cvt<T>::from_f(o_s[t * cols + c] * r * Cvt<T>::to_f(a.norm_w[c]));
      }
    }
  }
  float* to = OUT ? (last ? slot_state : nullptr) : a.carry + pc * elems;
  if (!OUT)
    for (int i = threadIdx.x; i < a.dim; i += blockDim.x) a.decay[pc * a.dim + i] = g_s[i];
  if (to) {
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
      const int row = (r >> 2) * 64 + rg * 4 + (r & 3);
      if (row >= a.dim) continue;
      float* p = to + (size_t)row * a.vdim + c0;
#pragma unroll
      for (int c = 0; c < 8; c += 4) {
        if (vec4) {
          if (c0 + c < a.vdim) *reinterpret_cast<float4*>(p + c) = make_float4(S[r][c], S[r][c + 1], S[r][c + 2], S[r][c + 3]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (c0 + c + j < a.vdim) p[c + j] = S[r][c + j];
        }
      }
    }
  }
}

// carry[p] = state in front of piece p:  S_0 = the sequence's state, S_(p+1) = decay_p * S_p + (state of piece p alone)
template <typename T>
__global__ void hgrn2_carry_kernel(const HgrnArgs<T> a) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, b = blockIdx.z;
  const int valid = a.new_lens ? a.new_lens[b] : a.s_new, base = a.seq_lens[b] - a.s_new;
  const int n = (valid + a.piece - 1) / a.piece;
  const int elems = a.dim * a.vdim;
  const float* state = a.state + ((size_t)a.slots[b] * a.heads + h) * elems;
  const size_t p0 = ((size_t)b * a.heads + h) * a.n_pieces;
  for (int e = blockIdx.x * blockDim.x + threadIdx.x; e < elems; e += gridDim.x * blockDim.x) {
    const int row = e / a.vdim;
    float S = base > 0 ? state[e] : 0.f;
    constexpr int G = 8;  // loads of a group are in flight together
    for (int p = 0; p < n; p += G) {
      float part[G], g[G];
#pragma unroll
      for (int i = 0; i < G; ++i)
        if (p + i < n - 1) { part[i] = __ldcg(a.carry + (p0 + p + i) * elems + e); g[i] = __ldcg(a.decay + (p0 + p + i) * a.dim + row); }
#pragma unroll
      for (int i = 0; i < G; ++i)
        if (p + i < n) {
          a.carry[(p0 + p + i) * elems + e] = S;
          if (p + i < n - 1) S = fmaf(g[i], S, part[i]);
        }
    }
  }
}

int round8(int v) { return (v + 7) / 8 * 8; }

template <typename T, int kRows, bool OUT, int kMaxThreads>
int hgrn2_launch_one(rb_ctx* ctx, const HgrnArgs<T>& a, int batch, int warps) {
  auto kern = hgrn2_kernel<T, kRows, OUT, kMaxThreads>;
  const int tokens = kTileTokens, dp = kRows * 16, cols = warps * 16;
  const size_t smem = (size_t)(tokens * (3 * dp + 2 * cols) + dp) * sizeof(float);
  static bool set[64] = {};  // the attribute belongs to the (kernel, device) pair
  const int dv = ctx->device & 63;
  if (!set[dv]) { RB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024)); set[dv] = true; }
  RB_CUDA(launch_kernel(kern, dim3((unsigned)a.n_pieces, (unsigned)a.heads, (unsigned)batch), dim3(warps * 32), smem, ctx->stream,
                        ctx->pdl, a));
  ctx->launches++;
  return RB_OK;
}

template <typename T, bool OUT>
int hgrn2_launch(rb_ctx* ctx, const HgrnArgs<T>& a, int batch) {
  const int warps = (a.vdim + 15) / 16;
  if (a.dim <= 64) return hgrn2_launch_one<T, 4, OUT, 512>(ctx, a, batch, warps);
  if (a.dim <= 128) return hgrn2_launch_one<T, 8, OUT, 512>(ctx, a, batch, warps);
  if (warps <= 8) return hgrn2_launch_one<T, 16, OUT, 256>(ctx, a, batch, warps);
  return hgrn2_launch_one<T, 16, OUT, 512>(ctx, a, batch, warps);
}

template <typename T>
int hgrn2_run(rb_ctx* ctx, HgrnArgs<T> a, int batch, int chunk) {
  // Pieces: enough blocks for about four per SM, none shorter than 64 tokens; one piece needs no second pass.
  int piece = chunk;
  if (piece <= 0) {
    const int want = std::max(1, (4 * ctx->sm_count) / std::max(1, batch * a.heads));
    piece = std::max(64, (a.s_new + want - 1) / want);
  }
  piece = (piece + kTileTokens - 1) / kTileTokens * kTileTokens;
  a.piece = piece;
  a.n_pieces = (a.s_new + piece - 1) / piece;
  if (a.n_pieces > 1) {
    const size_t elems = (size_t)a.dim * a.vdim, n = (size_t)batch * a.heads * a.n_pieces;
    const size_t bytes = n * (elems + a.dim) * sizeof(float);
    if (ctx->chunk_scratch_bytes < bytes) {
      float* fresh = nullptr;
      RB_CUDA(cudaMalloc(&fresh, bytes));
      if (ctx->chunk_scratch) ctx->retired.push_back(ctx->chunk_scratch);
      ctx->chunk_scratch = fresh;
      ctx->chunk_scratch_bytes = bytes;
    }
    a.carry = ctx->chunk_scratch;
    a.decay = ctx->chunk_scratch + n * elems;
    RB_TRY((hgrn2_launch<T, false>(ctx, a, batch)));
    const int blocks = (int)std::min<size_t>((elems + 255) / 256, 64);
    RB_CUDA(launch_kernel(hgrn2_carry_kernel<T>, dim3((unsigned)blocks, (unsigned)a.heads, (unsigned)batch), dim3(256), 0, ctx->stream,
                          ctx->pdl, a));
    ctx->launches++;
  }
  return hgrn2_launch<T, true>(ctx, a, batch);
}

template <typename T>
int conv_run(rb_ctx* ctx, ConvArgs<T> a, int batch) {
  const int C = a.qp + a.kp + a.vp;
  const size_t smem = (size_t)C * sizeof(float);
  auto kern = conv_norm_append_kernel<T>;
  static size_t set[64] = {};
  const int dv = ctx->device & 63;
  if (smem > 48 * 1024 && smem > set[dv]) {
    RB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    set[dv] = smem;
  }
  a.per_block = a.rows >= 16 * ctx->sm_count ? 8 : 1;
  const int blocks = (a.rows + a.per_block - 1) / a.per_block;
  RB_CUDA(launch_kernel(kern, dim3((unsigned)blocks), dim3(256), smem, ctx->stream, ctx->pdl, a));
  ctx->launches++;
  if (a.s_new > 1 && a.taps > 1) {
    RB_CUDA(launch_kernel(conv_ring_save_kernel<T>, dim3((unsigned)batch), dim3(256), 0, ctx->stream, ctx->pdl, a));
    ctx->launches++;
  }
  return RB_OK;
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
int add_norm_run(rb_ctx* ctx, const void* y, const float* acc, int n_acc, const void* gain, float eps, int64_t rows, int width, int ld,
                 float* h, void* x) {
  const int nchunk = ld / 8;
  const int threads = std::min(512, (nchunk + 31) / 32 * 32);
  const int chunks = (nchunk + threads - 1) / threads;
  const bool slabs = acc && n_acc > 0;
  // prefill: fewer blocks than rows, so that start-up is paid once per several rows
  const int64_t grid = std::min<int64_t>(rows, (int64_t)ctx->sm_count * (slabs ? 16 : std::max(4, 2048 / threads * 2)));
  auto go = [&](auto kern) -> int {
    RB_CUDA(launch_kernel(kern, dim3((unsigned)grid), dim3(threads), 0, ctx->stream, ctx->pdl, (const T*)y, acc, n_acc,
                          (size_t)rows * ld, (const T*)gain, eps, width, ld, h, (T*)x, rows));
    ctx->launches++;
    return RB_OK;
  };
  if (chunks <= 1) return slabs ? go(add_scaled_norm_kernel<T, 1, true>) : go(add_scaled_norm_kernel<T, 1, false>);
  if (chunks <= 2) return slabs ? go(add_scaled_norm_kernel<T, 2, true>) : go(add_scaled_norm_kernel<T, 2, false>);
  if (chunks <= 4) return slabs ? go(add_scaled_norm_kernel<T, 4, true>) : go(add_scaled_norm_kernel<T, 4, false>);
  return fail(RB_ERR_UNIMPLEMENTED, "rb_add_scaled_norm: width %d exceeds 16384", width);
}

}  // namespace

}  // namespace rb

using namespace rb;

extern "C" int32_t rb_embed_stream(rb_ctx* ctx, const void* table, int32_t dtype, int64_t vocab, int64_t width, int64_t ld,
                                   const uint32_t* ids, int64_t n_ids, float* h, void* x) {
  RB_REQUIRE(ctx && table && ids && h, "rb_embed_stream: null argument");
  RB_REQUIRE(vocab > 0 && width > 0 && ld >= width && (ld % 8) == 0, "rb_embed_stream: bad sizes");
  RB_REQUIRE(aligned16(table) && aligned16(h) && aligned16(x), "rb_embed_stream: buffers must be 16-byte aligned");
  if (n_ids == 0) return RB_OK;
  const double es = (double)dtype_size(dtype);
  ProfScope prof(ctx, RB_PROF_EMBED, (double)n_ids * width * (es + 4.0 + (x ? es : 0.0)), 0.0);
  const int threads = (int)std::min<int64_t>(256, (ld / 8 + 31) / 32 * 32);
  if (dtype == RB_BF16)
    RB_CUDA(launch_kernel(embed_stream_kernel<__nv_bfloat16>, dim3((unsigned)n_ids), dim3(threads), 0, ctx->stream, ctx->pdl,
                          (const __nv_bfloat16*)table, ids, vocab, (int)ld, h, (__nv_bfloat16*)x, ctx->status_dev));
  else if (dtype == RB_F32)
    RB_CUDA(launch_kernel(embed_stream_kernel<float>, dim3((unsigned)n_ids), dim3(threads), 0, ctx->stream, ctx->pdl,
                          (const float*)table, ids, vocab, (int)ld, h, (float*)x, ctx->status_dev));
  else
    return fail(RB_ERR_DTYPE, "rb_embed_stream: dtype %d unsupported", dtype);
  ctx->launches++;
  return RB_OK;
}

extern "C" int32_t rb_add_scaled_norm(rb_ctx* ctx, const void* y, const float* acc, int32_t n_acc, const void* gain, float eps,
                                      int64_t rows, int64_t width, int64_t ld, float* h, void* x, int32_t dtype) {
  RB_REQUIRE(ctx && gain && h && (y || (acc && n_acc > 0)), "rb_add_scaled_norm: null argument");
  RB_REQUIRE(rows >= 0 && width > 0 && ld >= width && (ld % 8) == 0, "rb_add_scaled_norm: bad sizes");
  RB_REQUIRE(aligned16(y) && aligned16(acc) && aligned16(h) && aligned16(x), "rb_add_scaled_norm: buffers must be 16-byte aligned");
  if (rows == 0) return RB_OK;
  if (!acc) n_acc = 0;
  const double es = (double)dtype_size(dtype);
  ProfScope prof(ctx, RB_PROF_NORM, (double)rows * width * ((y ? es : 0.0) + 4.0 * n_acc + 8.0 + (x ? es : 0.0)), 0.0);
  if (dtype == RB_BF16) return add_norm_run<__nv_bfloat16>(ctx, y, acc, n_acc, gain, eps, rows, (int)width, (int)ld, h, x);
  if (dtype == RB_F32) return add_norm_run<float>(ctx, y, acc, n_acc, gain, eps, rows, (int)width, (int)ld, h, x);
  return fail(RB_ERR_DTYPE, "rb_add_scaled_norm: dtype %d unsupported", dtype);
}

extern "C" int32_t rb_scalar_norm_rows(rb_ctx* ctx, const float* h, const int32_t* rows, int64_t row_step, const void* gain, float eps,
                                       int64_t n_rows, int64_t width, int64_t ld, void* out, int32_t dtype) {
  RB_REQUIRE(ctx && h && gain && out, "rb_scalar_norm_rows: null argument");
  RB_REQUIRE(n_rows >= 0 && width > 0 && ld >= width && (ld % 8) == 0 && (rows || row_step >= 1), "rb_scalar_norm_rows: bad sizes");
  RB_REQUIRE(aligned16(h) && aligned16(out), "rb_scalar_norm_rows: buffers must be 16-byte aligned");
  if (n_rows == 0) return RB_OK;
  const double es = (double)dtype_size(dtype);
  ProfScope prof(ctx, RB_PROF_NORM, (double)n_rows * width * (4.0 + es), 0.0);
  const int threads = (int)std::min<int64_t>(512, (ld / 8 + 31) / 32 * 32);
  if (dtype == RB_BF16)
    RB_CUDA(launch_kernel(scalar_norm_rows_kernel<__nv_bfloat16>, dim3((unsigned)n_rows), dim3(threads), 0, ctx->stream, ctx->pdl, h,
                          rows, row_step, (const __nv_bfloat16*)gain, eps, (int)width, (int)ld, (__nv_bfloat16*)out));
  else if (dtype == RB_F32)
    RB_CUDA(launch_kernel(scalar_norm_rows_kernel<float>, dim3((unsigned)n_rows), dim3(threads), 0, ctx->stream, ctx->pdl, h, rows,
                          row_step, (const float*)gain, eps, (int)width, (int)ld, (float*)out));
  else
    return fail(RB_ERR_DTYPE, "rb_scalar_norm_rows: dtype %d unsupported", dtype);
  ctx->launches++;
  return RB_OK;
}

extern "C" int32_t rb_conv_norm_append(rb_ctx* ctx, const void* src, const float* acc, int32_t n_acc, const void* bias,
                                       const void* conv, int32_t taps, const void* qw, const void* kw, float eps, int32_t batch,
                                       int32_t s_new, int32_t q_heads, int32_t kv_heads, int32_t key_dim, int32_t value_dim,
                                       int64_t src_ld, rb_kv_cache* c, int32_t layer, float* ring, const int32_t* new_lens,
                                       void* q_out, void* gate_out, int32_t dtype) {
  RB_REQUIRE(ctx && c && conv && q_out && (src || (acc && n_acc > 0)), "rb_conv_norm_append: null argument");
  RB_REQUIRE(taps >= 1 && (taps == 1 || ring), "rb_conv_norm_append: %d taps need the ring of earlier values", taps);
  RB_REQUIRE(batch > 0 && batch <= c->max_batch && s_new > 0, "rb_conv_norm_append: bad batch/seq");
  RB_REQUIRE(src || s_new == 1, "rb_conv_norm_append: split-K partials need single-token rows");
  RB_REQUIRE(q_heads > 0 && kv_heads >= 0 && key_dim > 0 && value_dim > 0 && key_dim <= c->head_dim && value_dim <= c->head_dim,
             "rb_conv_norm_append: bad head sizes");
  RB_REQUIRE(kv_heads == 0 || (kv_heads == c->kv_heads && layer >= 0 && layer < c->layers && dtype == c->dtype),
             "rb_conv_norm_append: the cache does not fit the layer");
  RB_REQUIRE(aligned16(src) && aligned16(acc) && aligned16(bias) && aligned16(conv) && aligned16(qw) && aligned16(kw) &&
                 aligned16(q_out) && aligned16(gate_out) && aligned16(ring),
             "rb_conv_norm_append: buffers must be 16-byte aligned");
  if (!acc) n_acc = 0;
  const int64_t rows = (int64_t)batch * s_new;
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    ConvArgs<T> a{};
    a.src = (const T*)src; a.acc = acc; a.n_acc = n_acc; a.acc_stride = (size_t)rows * src_ld;
    a.bias = (const T*)bias; a.conv = (const T*)conv; a.qw = (const T*)qw; a.kw = (const T*)kw;
    a.taps = taps; a.s_new = s_new; a.q_heads = q_heads; a.kv_heads = kv_heads; a.kd = key_dim; a.vd = value_dim; a.D = c->head_dim;
    a.qp = round8(q_heads * key_dim); a.kp = round8(kv_heads * key_dim); a.vp = round8(kv_heads * value_dim);
    a.gp = (int)src_ld - a.qp - a.kp - a.vp;
    RB_REQUIRE(a.gp >= 0 && (src_ld % 8) == 0, "rb_conv_norm_append: row pitch %lld does not hold the parts", (long long)src_ld);
    a.ld = src_ld; a.eps = eps;
    const size_t loff = (size_t)layer * c->layer_stride_elems();
    a.kc = kv_heads > 0 ? (T*)c->k + loff : nullptr;
    a.vc = kv_heads > 0 ? (T*)c->v + loff : nullptr;
    a.block_table = c->block_table; a.seq_lens = c->seq_lens; a.slots = c->slots; a.new_lens = new_lens;
    a.pages_per_seq = c->pages_per_seq; a.max_seq = c->max_seq; a.rows = (int)rows;
    a.ring = ring; a.q_out = (T*)q_out; a.gate_out = (T*)gate_out; a.status = ctx->status_dev;
    RB_REQUIRE((size_t)(a.qp + a.kp + a.vp) * sizeof(float) <= 200 * 1024, "rb_conv_norm_append: more than 51200 channels");
    const double C = a.qp + a.kp + a.vp, es = sizeof(T);
    ProfScope prof(ctx, RB_PROF_ROPE_KV, (double)rows * (src ? es * C : 4.0 * n_acc * src_ld) + rows * es * (C + (gate_out ? a.gp : 0)), 0.0);
    return conv_run<T>(ctx, a, batch);
  };
  if (dtype == RB_BF16) return fill(__nv_bfloat16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_conv_norm_append: dtype %d unsupported", dtype);
}

extern "C" int32_t rb_hgrn2(rb_ctx* ctx, const void* src, const float* acc, int32_t n_acc, int64_t src_ld, const void* f_bias,
                            const void* lower, const void* norm_w, float eps, int32_t heads, int32_t key_dim, int32_t value_dim,
                            int32_t batch, int32_t s_new, rb_kv_cache* c, const int32_t* new_lens, float* state, int32_t chunk,
                            void* out, int64_t out_ld, int32_t dtype) {
  RB_REQUIRE(ctx && c && f_bias && lower && norm_w && state && out && (src || (acc && n_acc > 0)), "rb_hgrn2: null argument");
  RB_REQUIRE(batch > 0 && batch <= c->max_batch && s_new > 0 && chunk >= 0, "rb_hgrn2: bad batch/seq");
  RB_REQUIRE(src || s_new == 1, "rb_hgrn2: split-K partials need single-token rows");
  RB_REQUIRE(heads > 0 && key_dim > 0 && value_dim > 0, "rb_hgrn2: bad head sizes");
  if (key_dim > 256 || value_dim > 256) return fail(RB_ERR_UNIMPLEMENTED, "rb_hgrn2: head sizes %d x %d exceed 256", key_dim, value_dim);
  RB_REQUIRE(aligned16(state), "rb_hgrn2: the state must be 16-byte aligned");
  if (!acc) n_acc = 0;
  const int64_t rows = (int64_t)batch * s_new;
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    HgrnArgs<T> a{};
    a.src = (const T*)src; a.acc = acc; a.n_acc = n_acc; a.acc_stride = (size_t)rows * src_ld;
    a.ld = src_ld; a.out_ld = out_ld;
    a.f_bias = (const T*)f_bias; a.lower = (const T*)lower; a.norm_w = (const T*)norm_w; a.eps = eps;
    a.heads = heads; a.dim = key_dim; a.vdim = value_dim;
    a.f_off = round8(heads * key_dim); a.v_off = 2 * a.f_off;
    RB_REQUIRE(src_ld >= a.v_off + heads * value_dim && out_ld >= (int64_t)heads * value_dim, "rb_hgrn2: row pitches too small");
    a.s_new = s_new; a.seq_lens = c->seq_lens; a.slots = c->slots; a.new_lens = new_lens; a.state = state; a.out = (T*)out;
    const double sb = 4.0 * key_dim * value_dim * heads, es = sizeof(T);
    ProfScope prof(ctx, RB_PROF_RECURRENCE,
                   2.0 * batch * sb + rows * ((src ? es : 4.0 * n_acc) * heads * (2.0 * key_dim + value_dim) + es * heads * value_dim),
                   5.0 * rows * heads * (double)key_dim * value_dim);
    return hgrn2_run<T>(ctx, a, batch, chunk);
  };
  if (dtype == RB_BF16) return fill(__nv_bfloat16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_hgrn2: dtype %d unsupported", dtype);
}
