// What attention of a pre-norm block needs from a fused input projection: head split, RMS norm of each query and key head,
// rotary positions, cache append; and the norm that follows the recurrence beside it (y times silu(z), over parts of a row).
// Single-token calls sum the projection's split-K slabs here.  All arithmetic is float32.
#include <math.h>

#include <algorithm>
#include <vector>

#include "recurrence.cuh"

namespace rb {

namespace {

template <typename T>
struct HeadArgs {
  const T* src;
  const float* acc;
  int n_acc;
  size_t acc_stride;
  const T* bias;
  int64_t ld;
  const T *qw, *kw;
  float eps;
  const float *cos_t, *sin_t;
  int half;                      // pairs that turn
  int s_new, rows, q_heads, kv_heads, kd, vd, D;
  int qp, kp, vp, gate, gp;      // padded widths of q, k, v; gate columns, and their padded number
  T *kc, *vc;
  const int32_t *block_table, *seq_lens;
  int pages_per_seq, max_seq;
  T *q_out, *gate_out;
  uint32_t* status;
};

__device__ __forceinline__ void store4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float* v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

// where row m's token sits; -1: outside the cache
template <typename T>
__device__ __forceinline__ int row_position(const HeadArgs<T>& a, int m) {
  const int pos = a.seq_lens[m / a.s_new] - a.s_new + m % a.s_new;
  if (pos >= 0 && pos < a.max_seq) return pos;
  if ((threadIdx.x & 31) == 0) { a.status[0] = (uint32_t)(-RB_ERR_INVALID); a.status[1] = 0x4EADu; a.status[2] = (uint32_t)pos; }
  return -1;
}
// (the kernel for any sizes)
template <typename T>
__device__ __forceinline__ T* cache_row(const HeadArgs<T>& a, T* cache, int m, int pos, int head) {
  const int page = a.block_table[(size_t)(m / a.s_new) * a.pages_per_seq + pos / kPageTokens];
  return cache + (((size_t)page * a.kv_heads + head) * kPageTokens + pos % kPageTokens) * a.D;
}

constexpr int kHeadWarps = 8;

// A team of kLanes lanes has one row and up to kHeads neighbouring query heads, key heads, value heads or pieces of the gate, so
// that weights, angles and the row's place in the cache are looked up once.  A lane has two quads of neighbouring elements of a
// head: one of the first half of the dimensions that turn and the quad it turns with, or two neighbouring quads of those that
// do not.
template <typename T, int kLanes, int kHeads, bool kSlabs>
__global__ void __launch_bounds__(kHeadWarps * 32, kSlabs ? 1 : 4) head_append_kernel(const HeadArgs<T> a) {
  constexpr int kTeams = kHeadWarps * 32 / kLanes, kPiece = kLanes * 8;   // teams of a block; columns of a gate piece
  pdl_launch_dependents();
  const int l = threadIdx.x % kLanes;
  const int nq = (a.q_heads + kHeads - 1) / kHeads, nk = (a.kv_heads + kHeads - 1) / kHeads;
  const int pieces = a.gate_out ? (a.gp + kPiece - 1) / kPiece : 0;
  const int m = (int)blockIdx.x * kTeams + (int)threadIdx.x / kLanes, group = blockIdx.y;
  // 0: query heads, 1: key heads, 2: value heads, 3: pieces of the gate
  const int kind = group < nq ? 0 : group < nq + nk ? 1 : group < nq + 2 * nk ? 2 : 3;
  const int h0 = kHeads * (kind == 0 ? group : kind == 1 ? group - nq : kind == 2 ? group - nq - nk : group - nq - 2 * nk);
  const int n = min(kHeads, (kind == 0 ? a.q_heads : kind < 3 ? a.kv_heads : pieces) - h0);
  const int size = kind < 2 ? a.kd : kind == 2 ? a.vd : kPiece;
  const int first = kind == 0 ? 0 : kind == 1 ? a.qp : kind == 2 ? a.qp + a.kp : a.qp + a.kp + a.vp;   // column of the part
  // the lane's two quads
  const int quads = kind < 2 ? a.half / 4 : 0, off = 2 * a.half + 8 * (l - quads);
  const bool turns = l < quads;
  const int c[2] = {turns ? 4 * l : kind < 2 ? off : 8 * l, turns ? 4 * l + a.half : kind < 2 ? off + 4 : 8 * l + 4};
  const T* norm = kind == 0 ? a.qw : kind == 1 ? a.kw : nullptr;
  float w[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
  for (int j = 0; j < 2; ++j)
    if (norm && c[j] < size) load4(norm + c[j], w[j]);
  pdl_wait();
  if (m >= a.rows) return;   // (the lanes of a team agree; nothing below crosses teams)
  const int b = (unsigned)m / (unsigned)a.s_new, pos = __ldg(a.seq_lens + b) - a.s_new + (m - b * a.s_new);
  float v[kHeads][2][4];
#pragma unroll
  for (int i = 0; i < kHeads; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int at = (h0 + i) * size + c[j];   // inside the part
#pragma unroll
      for (int e = 0; e < 4; ++e) v[i][j][e] = 0.f;
      if (i >= n || (kind < 3 ? c[j] >= size : at >= a.gp)) continue;
      if constexpr (!kSlabs) {
        load4(a.src + (size_t)m * a.ld + first + at, v[i][j]);
      } else {
        if (a.bias) load4(a.bias + first + at, v[i][j]);
        const float* p = a.acc + (size_t)m * a.ld + first + at;
        for (int k0 = 0; k0 < a.n_acc; k0 += 8) {   // slab order; the loads of up to eight slabs in flight together
          float t[8][4];
#pragma unroll
          for (int k = 0; k < 8; ++k)
            if (k0 + k < a.n_acc) load4(p + (size_t)(k0 + k) * a.acc_stride, t[k]);
#pragma unroll
          for (int k = 0; k < 8; ++k)
            if (k0 + k < a.n_acc) {
#pragma unroll
              for (int e = 0; e < 4; ++e) v[i][j][e] += t[k][e];
            }
        }
      }
    }
  if (kind == 3) {
#pragma unroll
    for (int i = 0; i < kHeads; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int at = (h0 + i) * kPiece + c[j];
        if (i < n && at < a.gp) store4(a.gate_out + (size_t)m * a.gp + at, v[i][j]);
      }
    return;
  }
  if (pos < 0 || pos >= a.max_seq) {
    if (l == 0) { a.status[0] = (uint32_t)(-RB_ERR_INVALID); a.status[1] = 0x4EADu; a.status[2] = (uint32_t)pos; }
    return;
  }
  float cs[4] = {1.f, 1.f, 1.f, 1.f}, sn[4] = {0.f, 0.f, 0.f, 0.f};
  if (turns) {
    load4(a.cos_t + (size_t)pos * a.half + c[0], cs);
    load4(a.sin_t + (size_t)pos * a.half + c[0], sn);
  }
  T* dst;
  int step = a.D;   // from a head to the next
  if (kind == 0) {
    dst = a.q_out + ((size_t)m * a.q_heads + h0) * a.D;
  } else {
    step *= kPageTokens;
    dst = (kind == 1 ? a.kc : a.vc) + (size_t)a.block_table[(size_t)b * a.pages_per_seq + pos / kPageTokens] * a.kv_heads * step +
          (size_t)h0 * step + pos % kPageTokens * a.D;
  }
  if (norm) {
    const uint32_t team = kLanes == 32 ? 0xffffffffu : ((1u << (kLanes & 31)) - 1u) << (threadIdx.x % 32 / kLanes * kLanes);
    const float inv = 1.0f / (float)size;
    float s[kHeads];
#pragma unroll
    for (int i = 0; i < kHeads; ++i) {
      s[i] = 0.f;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i] = fmaf(v[i][j][e], v[i][j][e], s[i]);
    }
#pragma unroll
    for (int o = kLanes / 2; o > 0; o >>= 1)
#pragma unroll
      for (int i = 0; i < kHeads; ++i) s[i] += __shfl_xor_sync(team, s[i], o);
#pragma unroll
    for (int i = 0; i < kHeads; ++i) {
      const float g = rsqrt_ftz(fmaf(s[i], inv, a.eps));
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) v[i][j][e] *= g * w[j][e];
    }
  }
#pragma unroll
  for (int i = 0; i < kHeads; ++i) {
    if (i >= n) break;
    if (turns) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float x = v[i][0][e], y = v[i][1][e];
        v[i][0][e] = fmaf(x, cs[e], -(y * sn[e]));
        v[i][1][e] = fmaf(y, cs[e], x * sn[e]);
      }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
      if (c[j] < a.D) store4(dst + (size_t)i * step + c[j], v[i][j]);   // (zeros beyond the head)
  }
}

// The same for any sizes: one warp per head and row, the head staged in shared memory.
template <typename T>
__global__ void __launch_bounds__(kHeadWarps * 32) head_append_any_kernel(const HeadArgs<T> a) {
  __shared__ float x_s[kHeadWarps][256];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int items = a.q_heads + 2 * a.kv_heads + (a.gate_out ? (a.gate + 255) / 256 : 0);
  const int64_t id = (int64_t)blockIdx.x * kHeadWarps + warp;
  const int item = (int)(id % items), m = (int)(id / items);
  if (m >= a.rows) return;
  const bool is_q = item < a.q_heads, is_k = !is_q && item < a.q_heads + a.kv_heads;
  const bool is_v = !is_q && !is_k && item < a.q_heads + 2 * a.kv_heads, is_gate = !is_q && !is_k && !is_v;
  const int head = is_q ? item : is_k ? item - a.q_heads : is_v ? item - a.q_heads - a.kv_heads : item - a.q_heads - 2 * a.kv_heads;
  const int size = is_q || is_k ? a.kd : is_v ? a.vd : min(256, a.gate - head * 256);
  const int col = is_q ? head * a.kd : is_k ? a.qp + head * a.kd : is_v ? a.qp + a.kp + head * a.vd : a.qp + a.kp + a.vp + head * 256;
  const T* norm = is_q ? a.qw : is_k ? a.kw : nullptr;
  float* x = x_s[warp];
  float s = 0.f;
  for (int i = lane; i < size; i += 32) {
    float v = a.src ? Cvt<T>::to_f(a.src[(size_t)m * a.ld + col + i]) : a.bias ? Cvt<T>::to_f(a.bias[col + i]) : 0.f;
    if (!a.src)
      for (int k = 0; k < a.n_acc; ++k) v += a.acc[(size_t)k * a.acc_stride + (size_t)m * a.ld + col + i];
    x[i] = v;
    s = fmaf(v, v, s);
  }
  if (is_gate) {
    for (int i = lane; i < size; i += 32) a.gate_out[(size_t)m * a.gp + head * 256 + i] = Cvt<T>::from_f(x[i]);
    return;
  }
  const int pos = row_position(a, m);
  if (pos < 0) return;
  if (norm) {
    const float g = 1.0f / sqrtf(warp_sum(s) / (float)size + a.eps);
    for (int i = lane; i < size; i += 32) x[i] *= g * Cvt<T>::to_f(norm[i]);
  }
  __syncwarp();
  T* dst = is_q ? a.q_out + ((size_t)m * a.q_heads + head) * a.D : cache_row(a, is_k ? a.kc : a.vc, m, pos, head);
  for (int i = lane; i < a.D; i += 32) {
    float y = i < size ? x[i] : 0.f;
    if (!is_v && i < 2 * a.half) {
      const bool first = i < a.half;
      const int f = first ? i : i - a.half;
      const float c = a.cos_t[(size_t)pos * a.half + f], sn = a.sin_t[(size_t)pos * a.half + f];
      y = first ? fmaf(y, c, -(x[i + a.half] * sn)) : fmaf(y, c, x[f] * sn);
    }
    dst[i] = Cvt<T>::from_f(y);
  }
}

// ------------------------------------------------------------------------------------------
// out = scale * weight * rms(y silu(z)), part by part of a row.  A part is one warp's or, kBlock, a whole block's; it stays in
// registers between the sum of squares and the scaling.  kVec: parts are 16-byte pieces.
// ------------------------------------------------------------------------------------------
template <typename T>
struct GroupNormArgs {
  const T* y;
  int64_t y_ld;
  const T* src;
  const float* acc;
  int n_acc;
  size_t acc_stride;
  int64_t ld;
  int col;
  const T* weight;
  int groups, part;
  float eps, scale;
  int64_t rows;
  T* out;
  int64_t out_ld;
};

template <typename T, int kChunks, bool kBlock, bool kVec, bool kSlabs>
__global__ void __launch_bounds__(kBlock ? 512 : 256) gated_norm_kernel(const GroupNormArgs<T> a) {
  constexpr bool kExact = sizeof(T) == 4;
  constexpr int E = kVec ? 8 : 1;   // elements of a piece
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t id = kBlock ? blockIdx.x : (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (id >= a.rows * a.groups) return;   // (a whole warp or block)
  const int me = kBlock ? threadIdx.x : threadIdx.x & 31, team = kBlock ? blockDim.x : 32;
  const int64_t row = id / a.groups;
  const int c0 = (int)(id % a.groups) * a.part;
  float v[kChunks][E];
  float s = 0.f;
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int i = (me + c * team) * E;
    if (i >= a.part) continue;
    float z[E];
    const size_t zi = (size_t)row * a.ld + a.col + c0 + i;
    if constexpr (kVec) {
      load8(a.y + row * a.y_ld + c0 + i, v[c]);
      if constexpr (!kSlabs) load8(a.src + zi, z);
      else {
#pragma unroll
        for (int e = 0; e < E; ++e) z[e] = 0.f;
        add_slabs<4>(a.acc, a.n_acc, a.acc_stride, zi, z);
      }
      silu8<kExact>(z);
    } else {
      v[c][0] = Cvt<T>::to_f(a.y[row * a.y_ld + c0 + i]);
      z[0] = kSlabs ? 0.f : Cvt<T>::to_f(a.src[zi]);
      for (int k = 0; k < a.n_acc; ++k) z[0] += a.acc[(size_t)k * a.acc_stride + zi];
      z[0] = silu_f<kExact>(z[0]);
    }
#pragma unroll
    for (int e = 0; e < E; ++e) { v[c][e] *= z[e]; s = fmaf(v[c][e], v[c][e], s); }
  }
  s = kBlock ? block_sum(s, red) : warp_sum(s);
  const float r = a.scale * rsqrt_ftz(s / (float)a.part + a.eps);
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int i = (me + c * team) * E;
    if (i >= a.part) continue;
    if constexpr (kVec) {
      float w[E];
      load8(a.weight + c0 + i, w);
#pragma unroll
      for (int e = 0; e < E; ++e) w[e] *= v[c][e] * r;
      store8(a.out + row * a.out_ld + c0 + i, w);
    } else {
      a.out[row * a.out_ld + c0 + i] = Cvt<T>::from_f(v[c][0] * r * Cvt<T>::to_f(a.weight[c0 + i]));
    }
  }
}

template <typename T>
int gated_norm_run(rb_ctx* ctx, const GroupNormArgs<T>& a, bool vec) {
  const int pieces = vec ? a.part / 8 : a.part;
  const int64_t parts = a.rows * a.groups;
  auto go = [&](auto kern, int threads, int64_t blocks) -> int {
    RB_REQUIRE(blocks <= 0x7fffffff, "rb_gated_group_norm: too many rows");
    RB_CUDA(launch_kernel(kern, dim3((unsigned)blocks), dim3(threads), 0, ctx->stream, ctx->pdl, a));
    ctx->launches++;
    return RB_OK;
  };
  auto pick = [&](auto vec_src, auto vec_slabs, auto src, auto slabs, int threads, int64_t blocks) {
    return go(vec ? (a.src ? vec_src : vec_slabs) : (a.src ? src : slabs), threads, blocks);
  };
#define RB_FORMS(chunks, block) gated_norm_kernel<T, chunks, block, true, false>, gated_norm_kernel<T, chunks, block, true, true>, \
                                gated_norm_kernel<T, chunks, block, false, false>, gated_norm_kernel<T, chunks, block, false, true>
  if (pieces <= 32) return pick(RB_FORMS(1, false), 256, (parts + 7) / 8);
  if (pieces <= 64) return pick(RB_FORMS(2, false), 256, (parts + 7) / 8);
  // a prompt's parts keep several loads per thread in flight; a few rows are latency, and want more threads
  const bool many = parts >= 4 * ctx->sm_count;
  const int want = many ? (pieces + 1) / 2 : pieces, threads = std::min(512, std::max(64, (want + 31) / 32 * 32));
  const int chunks = (pieces + threads - 1) / threads;
  if (chunks <= 1) return pick(RB_FORMS(1, true), threads, parts);
  if (chunks <= 2) return pick(RB_FORMS(2, true), threads, parts);
  if (chunks <= 4) return pick(RB_FORMS(4, true), threads, parts);
  if (!vec && chunks <= 32) return go(a.src ? gated_norm_kernel<T, 32, true, false, false> : gated_norm_kernel<T, 32, true, false, true>, threads, parts);
#undef RB_FORMS
  return fail(RB_ERR_UNIMPLEMENTED, "rb_gated_group_norm: parts of %d exceed 16384", a.part);
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
int round8(int v) { return (v + 7) / 8 * 8; }

template <typename T>
int head_append_run(rb_ctx* ctx, const HeadArgs<T>& a) {
  const bool quads = (a.kd % 4) == 0 && (a.vd % 4) == 0 && (a.half % 4) == 0;
  auto go = [&](auto kern, dim3 grid) -> int {
    RB_CUDA(launch_kernel(kern, grid, dim3(kHeadWarps * 32), 0, ctx->stream, ctx->pdl, a));
    ctx->launches++;
    return RB_OK;
  };
  if (!quads) {
    const int64_t warps = (int64_t)(a.q_heads + 2 * a.kv_heads + (a.gate_out ? (a.gate + 255) / 256 : 0)) * a.rows;
    RB_REQUIRE(warps <= 0x7fffffff, "rb_head_norm_rope_append: too many rows");
    return go(head_append_any_kernel<T>, dim3((unsigned)((warps + kHeadWarps - 1) / kHeadWarps)));
  }
  const bool few = a.rows < 4 * ctx->sm_count;
  auto pick = [&](auto slabs, auto one, auto four, int lanes) {
    const int at_once = a.acc || few ? 1 : 4, per = kHeadWarps * 32 / lanes;
    auto groups = [&](int n) { return (n + at_once - 1) / at_once; };
    const int gate = a.gate_out ? groups((a.gp + lanes * 8 - 1) / (lanes * 8)) : 0;
    const dim3 grid((unsigned)((a.rows + per - 1) / per), (unsigned)(groups(a.q_heads) + 2 * groups(a.kv_heads) + gate));
    return a.acc ? go(slabs, grid) : few ? go(one, grid) : go(four, grid);
  };
  if (a.D > 128) return pick(head_append_kernel<T, 32, 1, true>, head_append_kernel<T, 32, 1, false>, head_append_kernel<T, 32, 4, false>, 32);
  if (a.D > 64) return pick(head_append_kernel<T, 16, 1, true>, head_append_kernel<T, 16, 1, false>, head_append_kernel<T, 16, 4, false>, 16);
  return pick(head_append_kernel<T, 8, 1, true>, head_append_kernel<T, 8, 1, false>, head_append_kernel<T, 8, 4, false>, 8);
}

}  // namespace

}  // namespace rb

using namespace rb;

// amplitude * cos and sin of position * f[i], made in double precision
static int rotary_upload(rb_ctx* ctx, const std::vector<double>& f, int max_pos, double amplitude, float* cos_dev, float* sin_dev) {
  const size_t half = f.size();
  std::vector<float> c((size_t)max_pos * half), s((size_t)max_pos * half);
  for (int p = 0; p < max_pos; ++p)
    for (size_t i = 0; i < half; ++i) {
      c[(size_t)p * half + i] = (float)(amplitude * cos(p * f[i]));
      s[(size_t)p * half + i] = (float)(amplitude * sin(p * f[i]));
    }
  RB_CUDA(cudaMemcpyAsync(cos_dev, c.data(), c.size() * sizeof(float), cudaMemcpyHostToDevice, ctx->stream));
  RB_CUDA(cudaMemcpyAsync(sin_dev, s.data(), s.size() * sizeof(float), cudaMemcpyHostToDevice, ctx->stream));
  RB_CUDA(cudaStreamSynchronize(ctx->stream));  // the staging vectors die with this frame
  return RB_OK;
}

extern "C" int32_t rb_rotary_tables(rb_ctx* ctx, int32_t dims, int32_t max_pos, double base, double factor, double low, double high,
                                    double original, float* cos_dev, float* sin_dev) {
  RB_REQUIRE(ctx && cos_dev && sin_dev, "rb_rotary_tables: null argument");
  RB_REQUIRE(dims > 0 && (dims % 2) == 0 && max_pos > 0 && base > 0.0 && (original <= 0.0 || factor > 0.0), "rb_rotary_tables: bad sizes");
  const int half = dims / 2;
  std::vector<double> f(half);
  for (int i = 0; i < half; ++i) {
    f[i] = pow(base, -2.0 * i / dims);
    if (original <= 0.0) continue;
    const double turns = original * f[i] / (2.0 * 3.14159265358979323846);
    if (turns > high) continue;
    const double s = turns < low ? 0.0 : (turns - low) / (high - low);
    f[i] = (1.0 - s) * f[i] / factor + s * f[i];
  }
  return rotary_upload(ctx, f, max_pos, 1.0, cos_dev, sin_dev);
}

extern "C" int32_t rb_rotary_tables_yarn(rb_ctx* ctx, int32_t dims, int32_t max_pos, double base, double factor, double fast, double slow,
                                         double original, float* cos_dev, float* sin_dev) {
  RB_REQUIRE(ctx && cos_dev && sin_dev, "rb_rotary_tables_yarn: null argument");
  RB_REQUIRE(dims > 0 && (dims % 2) == 0 && max_pos > 0 && base > 0.0 && base != 1.0 && factor > 0.0 && fast > 0.0 && slow > 0.0 && original > 0.0,
             "rb_rotary_tables_yarn: bad sizes");
  const double two_pi = 2.0 * 3.14159265358979323846;
  auto index = [&](double turns) { return dims * log(original / (two_pi * turns)) / (2.0 * log(base)); };
  const double lo = std::max(floor(index(fast)), 0.0), hi = std::min(ceil(index(slow)), dims - 1.0);
  std::vector<double> f(dims / 2);
  for (int i = 0; i < dims / 2; ++i) {
    const double plain = pow(base, -2.0 * i / dims), stretch = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
    f[i] = plain / factor * stretch + plain * (1.0 - stretch);
  }
  return rotary_upload(ctx, f, max_pos, 0.1 * log(factor) + 1.0, cos_dev, sin_dev);
}

extern "C" int32_t rb_head_norm_rope_append(rb_ctx* ctx, const void* src, const float* acc, int32_t n_acc, const void* bias, int64_t src_ld,
                                            const void* qw, const void* kw, float eps, const float* cos_t, const float* sin_t,
                                            int32_t rot_dims, int32_t batch, int32_t s_new, int32_t q_heads, int32_t kv_heads,
                                            int32_t key_dim, int32_t value_dim, rb_kv_cache* c, int32_t layer, void* q_out, void* gate_out,
                                            int32_t gate_size, int32_t dtype) {
  RB_REQUIRE(ctx && c && q_out && (src || (acc && n_acc > 0)), "rb_head_norm_rope_append: null argument");
  RB_REQUIRE(batch > 0 && batch <= c->max_batch && s_new > 0, "rb_head_norm_rope_append: bad batch/seq");
  RB_REQUIRE(src || s_new == 1, "rb_head_norm_rope_append: split-K partials need single-token rows");
  RB_REQUIRE(q_heads > 0 && kv_heads == c->kv_heads && layer >= 0 && layer < c->layers && dtype == c->dtype && !c->shared(),
             "rb_head_norm_rope_append: the cache does not fit the layer");
  RB_REQUIRE(key_dim > 0 && value_dim > 0 && key_dim <= c->head_dim && value_dim <= c->head_dim && c->head_dim <= 256,
             "rb_head_norm_rope_append: bad head sizes");
  RB_REQUIRE(rot_dims >= 0 && rot_dims <= key_dim && (rot_dims % 2) == 0 && (rot_dims == 0 || (cos_t && sin_t)),
             "rb_head_norm_rope_append: %d of %d dimensions cannot turn", rot_dims, key_dim);
  RB_REQUIRE(aligned16(src) && aligned16(acc) && aligned16(bias) && aligned16(qw) && aligned16(kw) && aligned16(cos_t) && aligned16(sin_t) &&
                 aligned16(q_out) && aligned16(gate_out),
             "rb_head_norm_rope_append: buffers must be 16-byte aligned");
  const int64_t rows = (int64_t)batch * s_new;
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    HeadArgs<T> a{};
    a.src = (const T*)src; a.acc = src ? nullptr : acc; a.n_acc = src ? 0 : n_acc; a.acc_stride = (size_t)rows * src_ld;
    a.bias = (const T*)bias; a.ld = src_ld; a.qw = (const T*)qw; a.kw = (const T*)kw; a.eps = eps; a.cos_t = cos_t; a.sin_t = sin_t;
    a.half = rot_dims / 2; a.s_new = s_new; a.rows = (int)rows; a.q_heads = q_heads; a.kv_heads = kv_heads; a.kd = key_dim; a.vd = value_dim;
    a.D = c->head_dim; a.qp = round8(q_heads * key_dim); a.kp = round8(kv_heads * key_dim); a.vp = round8(kv_heads * value_dim);
    a.gate = gate_size; a.gp = round8(gate_size);
    RB_REQUIRE((src_ld % 8) == 0 && src_ld >= a.qp + a.kp + a.vp + (gate_out ? a.gp : 0) && (!gate_out || gate_size > 0),
               "rb_head_norm_rope_append: row pitch %lld does not hold the parts", (long long)src_ld);
    const size_t off = (size_t)layer * c->layer_stride_elems();
    a.kc = (T*)c->k + off; a.vc = (T*)c->v + off; a.block_table = c->block_table; a.seq_lens = c->seq_lens;
    a.pages_per_seq = c->pages_per_seq; a.max_seq = c->max_seq; a.q_out = (T*)q_out; a.gate_out = (T*)gate_out; a.status = ctx->status_dev;
    const double C = a.qp + a.kp + a.vp, es = sizeof(T);
    ProfScope prof(ctx, RB_PROF_ROPE_KV, (double)rows * ((src ? es : 4.0 * n_acc) * C + es * C), 0.0);
    return head_append_run<T>(ctx, a);
  };
  if (dtype == RB_BF16) return fill(__nv_bfloat16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_head_norm_rope_append: dtype %d unsupported", dtype);
}

extern "C" int32_t rb_gated_group_norm(rb_ctx* ctx, const void* y, int64_t y_ld, const void* src, const float* acc, int32_t n_acc,
                                       int64_t src_ld, int32_t col, const void* weight, int32_t groups, float eps, float scale,
                                       int64_t rows, int64_t width, void* out, int64_t out_ld, int32_t dtype) {
  RB_REQUIRE(ctx && y && weight && out && (src || (acc && n_acc > 0)), "rb_gated_group_norm: null argument");
  RB_REQUIRE(rows >= 0 && width > 0 && groups > 0 && width % groups == 0 && y_ld >= width && out_ld >= width && col >= 0 && src_ld >= col + width,
             "rb_gated_group_norm: bad sizes");
  if (rows == 0) return RB_OK;
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    GroupNormArgs<T> a{};
    a.y = (const T*)y; a.y_ld = y_ld; a.src = (const T*)src; a.acc = src ? nullptr : acc; a.n_acc = src ? 0 : n_acc;
    a.acc_stride = (size_t)rows * src_ld; a.ld = src_ld; a.col = col; a.weight = (const T*)weight; a.groups = groups;
    a.part = (int)(width / groups); a.eps = eps; a.scale = scale; a.rows = rows; a.out = (T*)out; a.out_ld = out_ld;
    const bool vec = (a.part % 8) == 0 && (y_ld % 8) == 0 && (src_ld % 8) == 0 && (col % 8) == 0 && (out_ld % 8) == 0 && aligned16(y) &&
                     aligned16(src) && aligned16(acc) && aligned16(weight) && aligned16(out);
    ProfScope prof(ctx, RB_PROF_NORM, (double)rows * width * (2.0 * sizeof(T) + (src ? sizeof(T) : 4.0 * n_acc)), 0.0);
    return gated_norm_run<T>(ctx, a, vec);
  };
  if (dtype == RB_BF16) return fill(__nv_bfloat16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_gated_group_norm: dtype %d unsupported", dtype);
}
