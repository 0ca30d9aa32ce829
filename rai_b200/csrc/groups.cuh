// Rows shared out among experts: where each expert's compact rows and work items start, from the experts' row counts.
#pragma once
#include "ctx.h"

namespace rb {

struct Groups {
  int item[kMaxExperts + 1], row[kMaxExperts + 1];
};

// By the whole block: E experts, tiles of `tile` rows, `per` items for each of them.
__device__ __forceinline__ void make_groups(Groups& g, const int32_t* count, int E, int tile, int per) {
  for (int e = threadIdx.x; e < E; e += blockDim.x) g.row[e + 1] = __ldcg(count + e);
  __syncthreads();
  if (threadIdx.x < 32) {
    int items = 0, rows = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + (int)threadIdx.x;
      const int c = e < E ? g.row[e + 1] : 0;
      int ri = c, ti = (c + tile - 1) / tile * per;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, ri, o), b = __shfl_up_sync(0xffffffffu, ti, o);
        if ((int)threadIdx.x >= o) { ri += a; ti += b; }
      }
      if (e < E) { g.row[e + 1] = rows + ri; g.item[e + 1] = items + ti; }
      rows += __shfl_sync(0xffffffffu, ri, 31);
      items += __shfl_sync(0xffffffffu, ti, 31);
    }
    if (threadIdx.x == 0) { g.row[0] = 0; g.item[0] = 0; }
  }
  __syncthreads();
}

// the e with start[e] <= at < start[e + 1]; at < start[E]
__device__ __forceinline__ int group_of(const int* start, int E, int at) {
  int lo = 0, hi = E;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (start[mid] <= at) lo = mid; else hi = mid;
  }
  return lo;
}

}  // namespace rb
