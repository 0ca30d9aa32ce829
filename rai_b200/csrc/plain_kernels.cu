// Plain CUDA-core kernels: the float32 data path (rai's F32 models), and a bf16 cross-check of the
// tensor-core kernels that a developer can select with RAI_B200_SIMPLE=1.  Straightforward
// shared-memory tiling, float32 accumulation, no tensor cores.
#include "ctx.h"

namespace rb {

// C[m, n] = sum_k X[m, k] * W[n, k]   (both operands K-major), epilogue as in rb_linear /
// rb_gated_linear.  64 x 64 output tile, 16-wide K slices, 256 threads with a 4 x 4 micro-tile.
template <typename T, bool GATED>
__global__ void gemm_plain_kernel(const T* __restrict__ x, const T* __restrict__ w, const T* __restrict__ w2,
                                  const T* __restrict__ bias, const T* __restrict__ residual, T* __restrict__ out,
                                  float* __restrict__ part, int m, int n, int k, int act, const T* __restrict__ act_params,
                                  int k_per_split) {
  constexpr int BM = 64, BN = 64, BK = 16;
  __shared__ float xs[BK][BM + 1];
  __shared__ float ws[BK][BN + 1];
  __shared__ float ws2[GATED ? BK : 1][BN + 1];
  const int tm = blockIdx.y * BM, tn = blockIdx.x * BN;
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  const int k0 = blockIdx.z * k_per_split, k1 = min(k, k0 + k_per_split);
  const float2 ac = act == RB_ACT_XIELU ? xielu_consts(act_params) : make_float2(0.f, 0.f);
  float acc[4][4] = {}, acc2[4][4] = {};
  for (int kk = k0; kk < k1; kk += BK) {
    for (int i = threadIdx.x; i < BM * BK; i += blockDim.x) {
      const int r = i / BK, c = i % BK;
      xs[c][r] = (tm + r < m && kk + c < k1) ? Cvt<T>::to_f(x[(size_t)(tm + r) * k + kk + c]) : 0.f;
      const bool ok = tn + r < n && kk + c < k1;
      ws[c][r] = ok ? Cvt<T>::to_f(w[(size_t)(tn + r) * k + kk + c]) : 0.f;
      if (GATED) ws2[c][r] = ok ? Cvt<T>::to_f(w2[(size_t)(tn + r) * k + kk + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < BK; ++c) {
      float a[4], b[4], b2[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = xs[c][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) { b[j] = ws[c][tx * 4 + j]; if (GATED) b2[j] = ws2[c][tx * 4 + j]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
          if (GATED) acc2[i][j] = fmaf(a[i], b2[j], acc2[i][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = tm + ty * 4 + i, c = tn + tx * 4 + j;
      if (r >= m || c >= n) continue;
      if (part) { part[((size_t)blockIdx.z * m + r) * n + c] = acc[i][j]; continue; }
      float v = acc[i][j];
      if (GATED) {
        // gate and up are tensors of the model dtype before the product (qwen2.rs:101-103)
        v = act_apply(act, v) * acc2[i][j];
      } else {
        if (bias) v += Cvt<T>::to_f(bias[c]);
        v = act_apply(act, v, ac);
        if (residual) v += Cvt<T>::to_f(residual[(size_t)r * n + c]);
      }
      out[(size_t)r * n + c] = Cvt<T>::from_f(v);
    }
}

// Decode-sized float32 Linear (M <= 8 rows; the reference's examples generate with batch 1 in float32,
// examples/qwen2/src/main.rs:58).  One warp per output feature: its weight row is read once with 16-byte loads
// and all M dot products ride along, so the kernel is bound by the weight stream like its bf16 counterpart.
template <bool GATED>
__global__ void __launch_bounds__(256) gemv_f32_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                       const float* __restrict__ w2, const float* __restrict__ bias,
                                                       const float* __restrict__ residual, float* __restrict__ out, int m,
                                                       int n, int k, int act, const float* __restrict__ act_params, int vec) {
  const float2 ac = act == RB_ACT_XIELU ? xielu_consts(act_params) : make_float2(0.f, 0.f);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col = blockIdx.x * 8 + warp;
  if (col >= n) return;
  const float* wr = w + (size_t)col * k;
  const float* wr2 = GATED ? w2 + (size_t)col * k : nullptr;
  float acc[8], acc2[8];
#pragma unroll
  for (int r = 0; r < 8; ++r) { acc[r] = 0.f; acc2[r] = 0.f; }
  if (vec) {
    for (int i = lane * 4; i < k; i += 128) {
      const float4 a = *reinterpret_cast<const float4*>(wr + i);
      float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
      if (GATED) b = *reinterpret_cast<const float4*>(wr2 + i);
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        if (r >= m) break;
        const float4 xv = *reinterpret_cast<const float4*>(x + (size_t)r * k + i);
        acc[r] = fmaf(a.w, xv.w, fmaf(a.z, xv.z, fmaf(a.y, xv.y, fmaf(a.x, xv.x, acc[r]))));
        if (GATED) acc2[r] = fmaf(b.w, xv.w, fmaf(b.z, xv.z, fmaf(b.y, xv.y, fmaf(b.x, xv.x, acc2[r]))));
      }
    }
  } else {
    for (int i = lane; i < k; i += 32) {
      const float a = wr[i], b = GATED ? wr2[i] : 0.f;
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        if (r >= m) break;
        const float xv = x[(size_t)r * k + i];
        acc[r] = fmaf(a, xv, acc[r]);
        if (GATED) acc2[r] = fmaf(b, xv, acc2[r]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    if (r >= m) break;
    float v = warp_sum(acc[r]);
    const float v2 = GATED ? warp_sum(acc2[r]) : 0.f;
    if (lane != 0) continue;
    if (GATED) {
      v = act_apply(act, v) * v2;
    } else {
      if (bias) v += bias[col];
      v = act_apply(act, v, ac);
      if (residual) v += residual[(size_t)r * n + col];
    }
    out[(size_t)r * n + col] = v;
  }
}

// One block per (token, query head): its 8 warps take every 8th key of the paged cache, each with an online
// softmax of its own (lanes split head_dim), and their (max, sum, O) states are merged through shared memory.
// float32 throughout.  Correct for any head_dim <= 32 * NJ.
constexpr int kPlainAttnWarps = 8;
template <typename T, int NJ>
__global__ void __launch_bounds__(kPlainAttnWarps * 32)
attention_plain_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                       const int32_t* __restrict__ block_table, const int32_t* __restrict__ seq_lens, int pages_per_seq,
                       int s_new, int q_heads, int kv_heads, int d, float scale, int window, T* __restrict__ out, int ext,
                       const AttnExtra x) {
  __shared__ float sm_m[kPlainAttnWarps], sm_l[kPlainAttnWarps], sm_o[kPlainAttnWarps][32 * NJ];
  const int m = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = m / s_new, s = m % s_new;
  const int limit = seq_lens[b] - s_new + s;  // last visible key
  const int kvh = h / (q_heads / kv_heads);
  float qv[NJ], o[NJ];
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int i = lane + 32 * j;
    qv[j] = i < d ? Cvt<T>::to_f(q[((size_t)m * q_heads + h) * d + i]) : 0.f;
    o[j] = 0.f;
  }
  float mx = -INFINITY, l = 0.f;
  const int call_base = seq_lens[b] - s_new;  // first token of this call
  const int first = ext ? first_visible(limit, x.window > 0 ? x.window : 1 << 30, x.chunk) : 0;
  const float slope = ext && x.alibi ? alibi_slope(h, q_heads) : 0.f;
  if (ext) scale *= query_temperature(limit, x.temp_every, x.temp_coef);
  for (int t = first + warp; t <= limit; t += kPlainAttnWarps) {
    // sliding window (qwen2.rs:316-334): it acts among the tokens of one call only, the cached prefix stays visible
    if (!ext && t >= call_base && t + window < limit) continue;
    const int page = block_table[(size_t)b * pages_per_seq + t / kPageTokens];
    const size_t off = (((size_t)page * kv_heads + kvh) * kPageTokens + (t % kPageTokens)) * d;
    float dot = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int i = lane + 32 * j;
      if (i < d) dot += qv[j] * Cvt<T>::to_f(k_cache[off + i]);
    }
    dot = warp_sum(dot) * scale;
    if (ext && x.softcap > 0.f) dot = x.softcap * tanhf(dot / x.softcap);
    dot = fmaf(-slope, (float)(limit - t), dot);
    const float mn = fmaxf(mx, dot);
    const float corr = expf(mx - mn), p = expf(dot - mn);
    l = l * corr + p;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int i = lane + 32 * j;
      if (i < d) o[j] = o[j] * corr + p * Cvt<T>::to_f(v_cache[off + i]);
    }
    mx = mn;
  }
  if (lane == 0) { sm_m[warp] = mx; sm_l[warp] = l; }
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int i = lane + 32 * j;
    if (i < d) sm_o[warp][i] = o[j];
  }
  __syncthreads();
  float M = -INFINITY;
#pragma unroll
  for (int w = 0; w < kPlainAttnWarps; ++w) M = fmaxf(M, sm_m[w]);
  float L = 0.f;
#pragma unroll
  for (int w = 0; w < kPlainAttnWarps; ++w) L += (sm_m[w] == -INFINITY) ? 0.f : sm_l[w] * expf(sm_m[w] - M);
  if (ext && x.sink) L += expf(Cvt<T>::to_f(((const T*)x.sink)[h]) - M);
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    float O = 0.f;
#pragma unroll
    for (int w = 0; w < kPlainAttnWarps; ++w) O += (sm_m[w] == -INFINITY) ? 0.f : sm_o[w][i] * expf(sm_m[w] - M);
    if (ext) {
      if (i >= x.value_dim) continue;
      const int col = h * x.value_dim + i;
      float y = O / L;
      if (x.gate) y *= sigmoid_f(Cvt<T>::to_f(((const T*)x.gate)[(size_t)m * x.gate_ld + (x.head_gate ? h : col)]));
      out[(size_t)m * x.out_ld + col] = Cvt<T>::from_f(y * x.out_scale);
    } else {
      out[((size_t)m * q_heads + h) * d + i] = Cvt<T>::from_f(O / L);
    }
  }
}

// The same where the heads' scores are mixed before the softmax: one block per token with all its heads, 32 keys at a time.
// Shared memory: q [heads][d], scores and weights [heads][33] each, max, sum and rescaling factor per head, O [heads][d].
constexpr int kTalkKeys = 32;
template <typename T>
__global__ void __launch_bounds__(256)
attention_talk_plain_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                            const int32_t* __restrict__ block_table, const int32_t* __restrict__ seq_lens, int pages_per_seq, int s_new,
                            int q_heads, int kv_heads, int d, float scale, T* __restrict__ out, const AttnExtra x) {
  extern __shared__ float smem_talk[];
  float* q_s = smem_talk;
  float* s_s = q_s + q_heads * d;
  float* p_s = s_s + q_heads * (kTalkKeys + 1);
  float* m_s = p_s + q_heads * (kTalkKeys + 1);
  float* l_s = m_s + q_heads;
  float* c_s = l_s + q_heads;
  float* o_s = c_s + q_heads;
  const int m = blockIdx.x, b = m / s_new, limit = seq_lens[b] - s_new + m % s_new, group = q_heads / kv_heads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const T* talk = (const T*)x.talk;
  for (int i = threadIdx.x; i < q_heads * d; i += blockDim.x) { q_s[i] = Cvt<T>::to_f(q[(size_t)m * q_heads * d + i]); o_s[i] = 0.f; }
  for (int h = threadIdx.x; h < q_heads; h += blockDim.x) { m_s[h] = -INFINITY; l_s[h] = 0.f; }
  const int first = first_visible(limit, x.window > 0 ? x.window : 1 << 30, x.chunk);
  for (int t0 = first / kTalkKeys * kTalkKeys; t0 <= limit; t0 += kTalkKeys) {
    const int page = block_table[(size_t)b * pages_per_seq + t0 / kPageTokens];
    auto row = [&](const T* cache, int kvh, int key) {
      return cache + (((size_t)page * kv_heads + kvh) * kPageTokens + (t0 + key) % kPageTokens) * d;
    };
    __syncthreads();
    for (int it = warp; it < q_heads * kTalkKeys; it += warps) {
      const int h = it / kTalkKeys, key = it % kTalkKeys;
      const T* kr = row(k_cache, h / group, key);
      float dot = 0.f;
      for (int i = lane; i < d; i += 32) dot = fmaf(q_s[h * d + i], Cvt<T>::to_f(kr[i]), dot);
      dot = warp_sum(dot);
      if (lane == 0) s_s[h * (kTalkKeys + 1) + key] = dot * scale;
    }
    __syncthreads();
    for (int h = warp; h < q_heads; h += warps) {   // a lane has a key
      float s = 0.f;
      for (int g = 0; g < q_heads; ++g) s = fmaf(Cvt<T>::to_f(talk[h * q_heads + g]), s_s[g * (kTalkKeys + 1) + lane], s);
      if (t0 + lane < first || t0 + lane > limit) s = -INFINITY;
      const float top = fmaxf(m_s[h], warp_max(s)), use = top == -INFINITY ? 0.f : top;
      const float p = expf(s - use), sum = warp_sum(p);
      p_s[h * (kTalkKeys + 1) + lane] = p;
      __syncwarp();
      if (lane == 0) { c_s[h] = expf(m_s[h] - use); l_s[h] = l_s[h] * c_s[h] + sum; m_s[h] = top; }
    }
    __syncthreads();
    for (int it = threadIdx.x; it < q_heads * x.value_dim; it += blockDim.x) {
      const int h = it / x.value_dim, i = it % x.value_dim;
      float o = o_s[h * d + i] * c_s[h];
      for (int key = 0; key < kTalkKeys; ++key) o = fmaf(p_s[h * (kTalkKeys + 1) + key], Cvt<T>::to_f(row(v_cache, h / group, key)[i]), o);
      o_s[h * d + i] = o;
    }
  }
  __syncthreads();
  for (int it = threadIdx.x; it < q_heads * x.value_dim; it += blockDim.x) {
    const int h = it / x.value_dim, i = it % x.value_dim;
    const float l = l_s[h] + (x.sink ? expf(Cvt<T>::to_f(((const T*)x.sink)[h]) - m_s[h]) : 0.f);
    out[(size_t)m * x.out_ld + it] = Cvt<T>::from_f(o_s[h * d + i] / l);
  }
}

static bool gemv_f32_launch(rb_ctx* ctx, const GemmArgs& a) {
  if (a.partials || a.m > 8) return false;
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const int vec = (a.k % 4 == 0) && al16(a.x) && al16(a.w) && (!a.w2 || al16(a.w2));
  const dim3 grid((unsigned)((a.n + 7) / 8));
  if (a.w2)
    gemv_f32_kernel<true><<<grid, 256, 0, ctx->stream>>>((const float*)a.x, (const float*)a.w, (const float*)a.w2, nullptr, nullptr,
                                                         (float*)a.out, (int)a.m, (int)a.n, (int)a.k, a.act, nullptr, vec);
  else
    gemv_f32_kernel<false><<<grid, 256, 0, ctx->stream>>>((const float*)a.x, (const float*)a.w, nullptr, (const float*)a.bias,
                                                          (const float*)a.residual, (float*)a.out, (int)a.m, (int)a.n, (int)a.k,
                                                          a.act, (const float*)a.act_params, vec);
  ctx->launches++;
  return true;
}

template <typename T>
static int gemm_plain_launch(rb_ctx* ctx, const GemmArgs& a) {
  const int splits = a.partials ? a.n_split : 1;
  dim3 grid((unsigned)((a.n + 63) / 64), (unsigned)((a.m + 63) / 64), (unsigned)splits);
  int kps = (int)a.k;
  if (splits > 1) kps = (int)(((a.k + splits - 1) / splits + 15) / 16 * 16);
  if (a.w2)
    gemm_plain_kernel<T, true><<<grid, 256, 0, ctx->stream>>>((const T*)a.x, (const T*)a.w, (const T*)a.w2, nullptr,
                                                             nullptr, (T*)a.out, nullptr, (int)a.m, (int)a.n, (int)a.k,
                                                             a.act, nullptr, kps);
  else
    gemm_plain_kernel<T, false><<<grid, 256, 0, ctx->stream>>>(
        (const T*)a.x, (const T*)a.w, nullptr, (const T*)a.bias, (const T*)a.residual, a.partials ? nullptr : (T*)a.out,
        a.partials ? (float*)a.out : nullptr, (int)a.m, (int)a.n, (int)a.k, a.act, (const T*)a.act_params, kps);
  ctx->launches++;
  return launch_status("gemm_plain");
}

int gemm_simple(rb_ctx* ctx, const GemmArgs& a, int dtype) {
  if (a.m == 0 || a.n == 0) return RB_OK;
  RB_REQUIRE(a.act != RB_ACT_XIELU || (a.act_params && !a.w2), "gemm: RB_ACT_XIELU needs its parameters and an ungated product");
  if (dtype == RB_F32) {
    if (gemv_f32_launch(ctx, a)) return launch_status("gemv_f32");
    return gemm_plain_launch<float>(ctx, a);
  }
  if (dtype == RB_BF16) return gemm_plain_launch<__nv_bfloat16>(ctx, a);
  return fail(RB_ERR_DTYPE, "gemm: dtype %d unsupported", dtype);
}

template <typename T, int NJ>
static int attention_plain_launch(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads, float scale,
                                  void* out, const AttnExtra* ext) {
  const size_t loff = (size_t)layer * c->layer_stride_elems();
  dim3 grid((unsigned)(batch * s_new), (unsigned)q_heads);
  attention_plain_kernel<T, NJ><<<grid, kPlainAttnWarps * 32, 0, ctx->stream>>>(
      (const T*)q, (const T*)c->k + loff, (const T*)c->v + loff, c->block_table, c->seq_lens, c->pages_per_seq, s_new, q_heads, c->kv_heads,
      c->head_dim, scale, c->window, (T*)out, ext ? 1 : 0, ext ? *ext : AttnExtra());
  ctx->launches++;
  return launch_status("attention_plain");
}

int attention_simple(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads,
                     float scale, void* out, int dtype, const AttnExtra* ext) {
  RB_REQUIRE(dtype == RB_F32 || dtype == RB_BF16, "attention: dtype %d unsupported", dtype);
  RB_REQUIRE(c->head_dim <= 1024, "attention: head_dim %d exceeds 1024", c->head_dim);
  const bool wide = c->head_dim > 256;
  const auto run = dtype == RB_F32 ? (wide ? attention_plain_launch<float, 32> : attention_plain_launch<float, 8>)
                                   : (wide ? attention_plain_launch<__nv_bfloat16, 32> : attention_plain_launch<__nv_bfloat16, 8>);
  return run(ctx, q, c, layer, batch, s_new, q_heads, scale, out, ext);
}

template <typename T>
static int talk_plain_launch(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads, float scale, void* out,
                             const AttnExtra& x) {
  const size_t loff = (size_t)layer * c->layer_stride_elems();
  const size_t smem = (size_t)q_heads * (2 * c->head_dim + 2 * (kTalkKeys + 1) + 3) * sizeof(float);
  if (smem > 200 * 1024) return fail(RB_ERR_UNIMPLEMENTED, "attention: %d mixed heads of %d exceed shared memory", q_heads, c->head_dim);
  auto kern = attention_talk_plain_kernel<T>;
  if (smem > 48 * 1024) RB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  kern<<<dim3((unsigned)(batch * s_new)), 256, smem, ctx->stream>>>((const T*)q, (const T*)c->k + loff, (const T*)c->v + loff, c->block_table,
                                                                   c->seq_lens, c->pages_per_seq, s_new, q_heads, c->kv_heads, c->head_dim,
                                                                   scale, (T*)out, x);
  ctx->launches++;
  return launch_status("attention_talk_plain");
}

int attention_talk_simple(rb_ctx* ctx, const void* q, rb_kv_cache* c, int layer, int batch, int s_new, int q_heads, float scale, void* out,
                          int dtype, const AttnExtra& x) {
  if (dtype == RB_F32) return talk_plain_launch<float>(ctx, q, c, layer, batch, s_new, q_heads, scale, out, x);
  if (dtype == RB_BF16) return talk_plain_launch<__nv_bfloat16>(ctx, q, c, layer, batch, s_new, q_heads, scale, out, x);
  return fail(RB_ERR_DTYPE, "attention: dtype %d unsupported", dtype);
}

}  // namespace rb
