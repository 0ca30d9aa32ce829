// The joints of blocks with a norm on both sides of a sublayer, on a float32 residual stream: x += norm(y), then optionally a
// weighted sum over the embedding and all layers' results so far, then the norm of the next sublayer's input.  A norm may run
// over equal parts of a row, each divided by its own root mean square.  All arithmetic is float32; a row stays in registers
// from the sublayer's output to the next one's input.
#include <algorithm>

#include "ctx.h"

namespace rb {

namespace {

template <typename T>
struct SandwichArgs {
  const T* y;
  const float* acc;
  int n_acc;
  size_t acc_stride;
  const T* post_gain;
  int groups, part;         // part: columns of one part of a row
  float eps;
  int64_t n_rows;
  int width, ld;
  const float* h_in;
  float* h_out;
  const T* depth;
  int n_depth;
  float* history;
  size_t history_stride;
  const T* gain;
  T* out;
  const int32_t* rows;      // rb_group_norm_rows: which rows (NULL with row_step: the last of every row_step)
  int64_t row_step;
};

// How the sums of squares of a row's parts come together: parts that are whole warps' pieces, whole 8-column chunks, or any
// columns.
enum { kWarpParts = 0, kChunkParts = 1, kAnyParts = 2 };

// 1 / rms of every part of the row whose chunks the block's threads hold in v (zeros beyond the row); r[c][i] receives the
// factor of element i of chunk c.  `buf` holds kWarpParts: a number per warp and c, kChunkParts: per chunk and per part,
// kAnyParts: per column and per part.
template <int kChunks, int kMode>
__device__ __forceinline__ void part_scales(const float (&v)[kChunks][8], int nchunk, int width, int part, int groups, float eps, float* buf,
                                            float (&r)[kChunks][kMode == kAnyParts ? 8 : 1]) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const float inv = 1.0f / (float)part;
  __syncthreads();   // the buffer may still be read from the last time
  float* sums = buf + (kMode == kAnyParts ? nchunk * 8 : nchunk);
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
    if (kMode == kAnyParts) {
      if (ch < nchunk) {
#pragma unroll
        for (int i = 0; i < 8; ++i) buf[ch * 8 + i] = v[c][i] * v[c][i];
      }
      continue;
    }
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s = fmaf(v[c][i], v[c][i], s);
    if (kMode == kChunkParts) {
      if (ch < nchunk) buf[ch] = s;
    } else {
      s = warp_sum(s);
      if (lane == 0) buf[c * warps + warp] = s;
    }
  }
  __syncthreads();
  if (kMode == kWarpParts) {
    const int per = part >> 8;   // entries of a part, in order of columns
#pragma unroll
    for (int c = 0; c < kChunks; ++c) {
      const int first = (c * warps + warp) / per * per;
      float s = 0.f;
      if (threadIdx.x + c * blockDim.x < nchunk)
        for (int k = 0; k < per; ++k) s += buf[first + k];
      r[c][0] = 1.0f / sqrtf(s * inv + eps);
    }
    return;
  }
  const int n = kMode == kChunkParts ? part >> 3 : part;
  for (int g = warp; g < groups; g += warps) {
    float s = 0.f;
    for (int k = lane; k < n; k += 32) s += buf[g * n + k];
    s = warp_sum(s);
    if (lane == 0) sums[g] = 1.0f / sqrtf(s * inv + eps);
  }
  __syncthreads();
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
    if (ch >= nchunk) continue;
    if (kMode == kChunkParts) r[c][0] = sums[ch / n];
    else {
#pragma unroll
      for (int i = 0; i < 8; ++i) r[c][i] = sums[min((ch * 8 + i) / part, groups - 1)];
    }
  }
}

template <typename T, int kChunks, int kMode, bool kSlabs>
__global__ void __launch_bounds__(512) sandwich_kernel(const SandwichArgs<T> a) {
  extern __shared__ float buf[];
  pdl_launch_dependents();
  const int nchunk = a.ld >> 3;
  pdl_wait();
  const bool adds = a.y || kSlabs;
  for (int64_t row = blockIdx.x; row < a.n_rows; row += gridDim.x) {
    const int64_t from = a.rows ? a.rows[row] : a.row_step > 0 ? (row + 1) * a.row_step - 1 : row;
    const size_t base = (size_t)row * a.ld, in = (size_t)from * a.ld;
    float x[kChunks][8], r[kChunks][kMode == kAnyParts ? 8 : 1];
    if (adds) {
      float v[kChunks][8];
#pragma unroll
      for (int c = 0; c < kChunks; ++c) {
        const int ch = threadIdx.x + c * blockDim.x;
#pragma unroll
        for (int i = 0; i < 8; ++i) v[c][i] = 0.f;
        if (ch >= nchunk) continue;
        if (a.y) load8(a.y + base + ch * 8, v[c]);
        if (kSlabs) add_slabs<(kChunks > 1 ? 4 : 8)>(a.acc, a.n_acc, a.acc_stride, base + ch * 8, v[c]);
        load8(a.h_in + in + ch * 8, x[c]);
      }
      part_scales<kChunks, kMode>(v, nchunk, a.width, a.part, a.groups, a.eps, buf, r);
#pragma unroll
      for (int c = 0; c < kChunks; ++c) {
        const int ch = threadIdx.x + c * blockDim.x;
        if (ch >= nchunk) continue;
        float g[8];
        load8(a.post_gain + ch * 8, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) x[c][i] = fmaf(v[c][i] * r[c][kMode == kAnyParts ? i : 0], g[i], x[c][i]);
      }
    } else {
#pragma unroll
      for (int c = 0; c < kChunks; ++c) {
        const int ch = threadIdx.x + c * blockDim.x;
        if (ch < nchunk) load8(a.h_in + in + ch * 8, x[c]);
      }
    }
#pragma unroll
    for (int c = 0; c < kChunks; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch >= nchunk) {
#pragma unroll
        for (int i = 0; i < 8; ++i) x[c][i] = 0.f;
        continue;
      }
      if (a.n_depth > 0) {
        float* hist = a.history + base + ch * 8;
        const int last = a.n_depth - 1;
        store8(hist + (size_t)last * a.history_stride, x[c]);
        float s[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) s[i] = 0.f;
        for (int j0 = 0; j0 < last; j0 += 4) {   // the loads of four earlier results in flight together
          float t[4][8], w[4];
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (j0 + j < last) {
              w[j] = Cvt<T>::to_f(a.depth[j0 + j]);
              load8(hist + (size_t)(j0 + j) * a.history_stride, t[j]);
            }
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (j0 + j < last) {
#pragma unroll
              for (int i = 0; i < 8; ++i) s[i] = fmaf(w[j], t[j][i], s[i]);
            }
        }
        const float w = Cvt<T>::to_f(a.depth[last]);
#pragma unroll
        for (int i = 0; i < 8; ++i) x[c][i] = fmaf(w, x[c][i], s[i]);
      }
      if (a.h_out) store8(a.h_out + base + ch * 8, x[c]);
    }
    if (!a.out) continue;
    part_scales<kChunks, kMode>(x, nchunk, a.width, a.part, a.groups, a.eps, buf, r);
#pragma unroll
    for (int c = 0; c < kChunks; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch >= nchunk) continue;
      float g[8];
      load8(a.gain + ch * 8, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) g[i] *= x[c][i] * r[c][kMode == kAnyParts ? i : 0];
      store8(a.out + base + ch * 8, g);
    }
  }
}

template <typename T>
int sandwich_run(rb_ctx* ctx, SandwichArgs<T> a) {
  const int nchunk = a.ld / 8;
  const int threads = std::min(512, (nchunk + 31) / 32 * 32), chunks = (nchunk + threads - 1) / threads;
  const bool slabs = a.n_acc > 0;
  const int mode = (a.part % 256) == 0 && a.ld == a.width ? kWarpParts : (a.part % 8) == 0 ? kChunkParts : kAnyParts;
  const size_t smem = (size_t)((mode == kAnyParts ? a.ld : std::max(nchunk, chunks * threads / 32)) + a.groups) * sizeof(float);
  const int64_t grid = std::min<int64_t>(a.n_rows, (int64_t)ctx->sm_count * (slabs ? 16 : std::max(4, 2048 / threads * 2)));
  auto go = [&](auto kern) -> int {
    if (smem > 48 * 1024) RB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    RB_CUDA(launch_kernel(kern, dim3((unsigned)grid), dim3(threads), smem, ctx->stream, ctx->pdl, a));
    ctx->launches++;
    return RB_OK;
  };
  auto pick = [&](auto n) -> int {
    constexpr int K = decltype(n)::value;
    if (mode == kWarpParts) return slabs ? go(sandwich_kernel<T, K, kWarpParts, true>) : go(sandwich_kernel<T, K, kWarpParts, false>);
    if (mode == kChunkParts) return slabs ? go(sandwich_kernel<T, K, kChunkParts, true>) : go(sandwich_kernel<T, K, kChunkParts, false>);
    return slabs ? go(sandwich_kernel<T, K, kAnyParts, true>) : go(sandwich_kernel<T, K, kAnyParts, false>);
  };
  if (chunks <= 1) return pick(std::integral_constant<int, 1>());
  if (chunks <= 2) return pick(std::integral_constant<int, 2>());
  if (chunks <= 4) return pick(std::integral_constant<int, 4>());
  return fail(RB_ERR_UNIMPLEMENTED, "rb_sandwich_join: width %d exceeds 16384", a.width);
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

int sandwich_join(rb_ctx* ctx, const SandwichSpec& s, int dtype) {
  const bool adds = s.y || (s.acc && s.n_acc > 0);
  RB_REQUIRE(ctx && s.h_in && (!adds || s.post_gain) && (!s.out || s.gain) && (s.n_depth <= 0 || (s.depth && s.history)),
             "rb_sandwich_join: null argument");
  RB_REQUIRE(s.rows >= 0 && s.width > 0 && s.ld >= s.width && (s.ld % 8) == 0 && s.groups > 0 && s.width % s.groups == 0 && s.n_depth >= 0,
             "rb_sandwich_join: bad sizes");
  RB_REQUIRE(aligned16(s.y) && aligned16(s.acc) && aligned16(s.post_gain) && aligned16(s.h_in) && aligned16(s.h_out) && aligned16(s.history) &&
                 (s.history_stride % 4) == 0 && aligned16(s.gain) && aligned16(s.out),
             "rb_sandwich_join: buffers must be 16-byte aligned");
  if (s.rows == 0) return RB_OK;
  const double es = (double)dtype_size(dtype);
  ProfScope prof(ctx, RB_PROF_NORM,
                 (double)s.rows * s.width * ((s.y ? es : 0.0) + (s.acc ? 4.0 * s.n_acc : 0.0) + 4.0 + (s.h_out ? 4.0 : 0.0) + 4.0 * s.n_depth +
                                             (s.out ? es : 0.0)), 0.0);
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    SandwichArgs<T> a{};
    a.y = (const T*)s.y; a.acc = s.acc; a.n_acc = s.acc ? s.n_acc : 0; a.acc_stride = (size_t)s.rows * s.ld; a.post_gain = (const T*)s.post_gain;
    a.groups = s.groups; a.part = s.width / s.groups; a.eps = s.eps; a.n_rows = s.rows; a.width = s.width; a.ld = s.ld; a.h_in = s.h_in;
    a.h_out = s.h_out; a.depth = (const T*)s.depth; a.n_depth = s.n_depth; a.history = s.history; a.history_stride = (size_t)s.history_stride;
    a.gain = (const T*)s.gain; a.out = (T*)s.out;
    return sandwich_run<T>(ctx, a);
  };
  if (dtype == RB_BF16) return fill(__nv_bfloat16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_sandwich_join: dtype %d unsupported", dtype);
}

}  // namespace rb

using namespace rb;

extern "C" int32_t rb_sandwich_join(rb_ctx* ctx, const void* y, const float* acc, int32_t n_acc, const void* post_gain, int32_t groups,
                                    float eps, int64_t rows, int64_t width, int64_t ld, const float* h_in, float* h_out, const void* depth,
                                    int32_t n_depth, float* history, int64_t history_stride, const void* gain, void* out, int32_t dtype) {
  SandwichSpec s;
  s.y = y; s.acc = acc; s.n_acc = acc ? n_acc : 0; s.post_gain = post_gain; s.groups = groups; s.eps = eps; s.rows = rows;
  s.width = (int)width; s.ld = (int)ld; s.h_in = h_in; s.h_out = h_out; s.depth = depth; s.n_depth = depth ? n_depth : 0;
  s.history = history; s.history_stride = history_stride; s.gain = gain; s.out = out;
  return sandwich_join(ctx, s, dtype);
}

extern "C" int32_t rb_group_norm_rows(rb_ctx* ctx, const float* h, const int32_t* rows, int64_t row_step, const void* gain, int32_t groups,
                                      float eps, int64_t n_rows, int64_t width, int64_t ld, void* out, int32_t dtype) {
  RB_REQUIRE(ctx && h && gain && out, "rb_group_norm_rows: null argument");
  RB_REQUIRE(n_rows >= 0 && width > 0 && ld >= width && (ld % 8) == 0 && groups > 0 && width % groups == 0 && (rows || row_step >= 1),
             "rb_group_norm_rows: bad sizes");
  RB_REQUIRE(aligned16(h) && aligned16(out) && aligned16(gain), "rb_group_norm_rows: buffers must be 16-byte aligned");
  if (n_rows == 0) return RB_OK;
  ProfScope prof(ctx, RB_PROF_NORM, (double)n_rows * width * (4.0 + dtype_size(dtype)), 0.0);
  auto fill = [&](auto tag) -> int {
    using T = decltype(tag);
    SandwichArgs<T> a{};
    a.groups = groups; a.part = (int)(width / groups); a.eps = eps; a.n_rows = n_rows; a.width = (int)width; a.ld = (int)ld; a.h_in = h;
    a.gain = (const T*)gain; a.out = (T*)out; a.rows = rows; a.row_step = row_step;
    return sandwich_run<T>(ctx, a);
  };
  if (dtype == RB_BF16) return fill(__nv_bfloat16());
  if (dtype == RB_F32) return fill(float());
  return fail(RB_ERR_DTYPE, "rb_group_norm_rows: dtype %d unsupported", dtype);
}
