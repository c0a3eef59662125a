// Which tile of queries of a packed batch a CTA works on.
#pragma once
#include "common.cuh"

namespace mv {

// Tile blockIdx.x of the batch, tiles of `rows` queries, those of a sequence in descending order: s_tile[0] = its sequence (-1: none),
// s_tile[1] = its number within it.  All kThreads threads; s_scan has one int per warp.
template <int kThreads>
__device__ __forceinline__ void find_query_tile(const int32_t* cu_q, int num_seqs, int rows, int* s_tile, int* s_scan) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid == 0) {
    s_tile[0] = -1;
    s_tile[1] = 0;
  }
  __syncthreads();
  int carry = 0;
  for (int base = 0; base < num_seqs; base += kThreads) {
    const int s = base + tid;
    int n = 0;
    if (s < num_seqs) n = (max(cu_q[s + 1] - cu_q[s], 0) + rows - 1) / rows;
    int incl = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += v;
    }
    if (lane == 31) s_scan[warp] = incl;
    __syncthreads();
    int before = 0, tot = 0;
    for (int w = 0; w < kThreads / 32; ++w) {
      if (w < warp) before += s_scan[w];
      tot += s_scan[w];
    }
    const int start = carry + before + incl - n, x = static_cast<int>(blockIdx.x);
    if (n > 0 && x >= start && x < start + n) { s_tile[0] = s; s_tile[1] = n - 1 - (x - start); }
    carry += tot;
    __syncthreads();
  }
}

// Tile x of the same order, by every warp for itself: false without a tile.
__device__ __forceinline__ bool find_query_tile_warp(const int32_t* cu_q, int num_seqs, int rows, int x, int& seq, int& tile) {
  const int lane = threadIdx.x & 31;
  int base = 0;
  for (int b = 0; b < num_seqs; b += 32) {
    const int s = b + lane, n = s < num_seqs ? (max(cu_q[s + 1] - cu_q[s], 0) + rows - 1) / rows : 0;
    int incl = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += v;
    }
    const uint32_t past = __ballot_sync(0xffffffffu, base + incl > x);
    if (past) {
      const int at = __ffs(past) - 1;
      seq = b + at;
      tile = base + __shfl_sync(0xffffffffu, incl, at) - 1 - x;
      return true;
    }
    base += __shfl_sync(0xffffffffu, incl, 31);
  }
  return false;
}

}  // namespace mv
