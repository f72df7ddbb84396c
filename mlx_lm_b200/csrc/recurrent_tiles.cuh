// What the recurrences that run in tiles of rows on tensor cores share: how long a request's run of rows is, and staging of
// one head's rows in shared memory.
#pragma once

#include "common.cuh"

// Rows t0 .. t1-1 that belong to request r (they come first in the range).  Every thread of the block calls it.
__device__ __forceinline__ int run_length(const int* __restrict__ token_req, int t0, int t1, int r) {
  int n = 0;
  for (int base = t0; base < t1; base += blockDim.x) {
    const int t = base + threadIdx.x;
    n += __syncthreads_count(t < t1 && token_req[t] == r);
  }
  return n;
}

// Rows of v: columns v0 .. v0 + VS - 1 of one head into [rows, lds]; zeros beyond n rows and beyond V columns.
template <bool VEC>
__device__ __forceinline__ void stage_values(const __nv_bfloat16* src, int ld, int row0, int n, int rows, int v0, int V, int VS,
                                             __nv_bfloat16* sv, int lds) {
  if (VEC) {
    const int per = VS / 8;
#pragma unroll 4
    for (int e = threadIdx.x; e < rows * per; e += blockDim.x) {
      const int tok = e / per, c = (e - tok * per) * 8;
      uint4 u = make_uint4(0u, 0u, 0u, 0u);
      if (tok < n && v0 + c < V) u = *reinterpret_cast<const uint4*>(src + (size_t)(row0 + tok) * ld + v0 + c);
      *reinterpret_cast<uint4*>(sv + tok * lds + c) = u;
    }
  } else {
    for (int e = threadIdx.x; e < rows * VS; e += blockDim.x) {
      const int tok = e / VS, c = e - tok * VS;
      sv[tok * lds + c] = (tok < n && v0 + c < V) ? src[(size_t)(row0 + tok) * ld + v0 + c] : __float2bfloat16_rn(0.f);
    }
  }
}
