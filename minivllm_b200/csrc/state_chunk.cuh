// Chunked forms of the matrix-state recurrences (state_scan.cuh) for prompts, bf16 operands on tensor cores, fp32 state.
//
// A first kernel works on all chunks of 64 tokens at once and leaves in scratch what does not depend on the state.  A
// second one walks a sequence's chunks with the state in registers.  It computes everything transposed: a warp owns 16
// columns of the state as the 16 rows of m16n8k16 accumulators, and an accumulator's layout is that of the A operand of
// the next product, so that state, right-hand sides and results go from product to product without leaving the
// registers, and warps share nothing but the tiles they read (two stages of cp.async).
//
// What the recurrence forms itself (the state among it) is fp32 and enters a product as two bf16 terms, value and rounding
// residue; outputs of projections and convolutions enter as they are.
#pragma once
#include <algorithm>
#include "mma.cuh"
#include "state_scan.cuh"

namespace mv {

constexpr int kChunk = 64;
constexpr int kCkRow = kChunk + 8;              // row stride of a 64 x 64 tile in shared memory
constexpr float kLog2e = 1.4426950408889634f;
using Mma = Mma16816<__nv_bfloat16>;

inline int64_t chunk_bound(int64_t tokens, int num_seqs) { return tokens / kChunk + std::min<int64_t>(num_seqs, tokens); }

// Chunks of the sequences before s.  Whole warp.
__device__ __forceinline__ int chunks_before(const int32_t* cu, int s) {
  int n = 0;
  for (int i = threadIdx.x & 31; i < s; i += 32) n += (max(cu[i + 1] - cu[i], 0) + kChunk - 1) / kChunk;
  return __reduce_add_sync(0xffffffffu, n);
}
// Sequence and chunk within it of the x-th chunk of the batch; false past the last.  Whole warp.
__device__ __forceinline__ bool find_chunk(const int32_t* cu, int num_seqs, int x, int& seq, int& chunk) {
  const int lane = threadIdx.x & 31;
  int base = 0;
  for (int b = 0; b < num_seqs; b += 32) {
    const int s = b + lane, n = s < num_seqs ? (max(cu[s + 1] - cu[s], 0) + kChunk - 1) / kChunk : 0;
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
      chunk = x - base - __shfl_sync(0xffffffffu, incl - n, at);
      return true;
    }
    base += __shfl_sync(0xffffffffu, incl, 31);
  }
  return false;
}

// The lane's part of ldmatrix addresses (in elements): a 16 x 16 block as two n-tiles of a B operand with the reduction
// along a row, and along a column (.trans).  The first form with .trans also reads a transposed A operand.
struct LaneAt {
  int row_b, col_b, row_t, col_t;
  __device__ __forceinline__ explicit LaneAt(int lane) {
    const int l7 = lane & 7, l8 = (lane >> 3) & 1, l16 = lane >> 4;
    row_b = l7 + l16 * 8; col_b = l8 * 8;
    row_t = l7 + l8 * 8; col_t = l16 * 8;
  }
};

// The 16 columns of a warp: tile n holds channels 8 n .. 8 n + 7 (accumulator columns), rows are value columns.
template <int K> struct ChunkState {
  float s[K / 8][4];
  // gS: the head's (K, V) state; columns v0 .. v0 + 15 below v_end
  __device__ __forceinline__ void load(const float* gS, int v0, int v_end, int V, int K_real, int lane, bool on) {
    const int g = lane >> 2, c2 = (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < K / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int ch = n * 8 + c2 + (e & 1), v = v0 + g + (e >> 1) * 8;
        s[n][e] = on && ch < K_real && v < v_end ? gS[static_cast<int64_t>(ch) * V + v] : 0.f;
      }
  }
  __device__ __forceinline__ void store(float* gS, int v0, int v_end, int V, int K_real, int lane) const {
    const int g = lane >> 2, c2 = (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < K / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int ch = n * 8 + c2 + (e & 1), v = v0 + g + (e >> 1) * 8;
        if (ch < K_real && v < v_end) gS[static_cast<int64_t>(ch) * V + v] = s[n][e];
      }
  }
};

// Two adjacent accumulator tiles as both terms of an A operand.
__device__ __forceinline__ void split_a(const float (&x)[4], const float (&y)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  split2(x[0], x[1], hi[0], lo[0]);
  split2(x[2], x[3], hi[1], lo[1]);
  split2(y[0], y[1], hi[2], lo[2]);
  split2(y[2], y[3], hi[3], lo[3]);
}

// acc += A B^T for a lower-triangular 64 x 64 B in two terms (rows of kCkRow elements, the second 64 rows after the
// first), A's 16-column block ib.  Here and below two tiles' products alternate, so that a product rarely waits for the
// one before it.
template <bool kTwoA>
__device__ __forceinline__ void mma_lower(float (&acc)[8][4], const uint32_t (&hi)[4], const uint32_t (&lo)[4], uint32_t b_smem,
                                          int ib, const LaneAt& at) {
#pragma unroll
  for (int n0 = 0; n0 < 4; n0 += 2) {
    uint32_t b[2][4];
    const uint32_t addr = b_smem + ((n0 * 16 + at.row_b) * kCkRow + ib * 16 + at.col_b) * 2;
#pragma unroll
    for (int j = 0; j < 2; ++j)
      if (n0 + j >= ib) {
        ldmatrix_x4(b[j], addr + j * 16 * kCkRow * 2);
        Mma::run(acc[2 * (n0 + j)], hi, b[j][0], b[j][1]);
        Mma::run(acc[2 * (n0 + j) + 1], hi, b[j][2], b[j][3]);
      }
    if (kTwoA) {
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (n0 + j >= ib) {
          Mma::run(acc[2 * (n0 + j)], lo, b[j][0], b[j][1]);
          Mma::run(acc[2 * (n0 + j) + 1], lo, b[j][2], b[j][3]);
        }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
      if (n0 + j >= ib) {
        ldmatrix_x4(b[j], addr + (j * 16 + kChunk) * kCkRow * 2);
        Mma::run(acc[2 * (n0 + j)], hi, b[j][0], b[j][1]);
        Mma::run(acc[2 * (n0 + j) + 1], hi, b[j][2], b[j][3]);
      }
  }
}

// cp.async of the blocks on and below the diagonal of a 64 x 64 tile (both terms) into rows of kCkRow elements.
__device__ __forceinline__ void load_lower(uint32_t dst, const __nv_bfloat16* src, int tid, int threads) {
  for (int i = tid; i < 2 * kChunk * 8; i += threads) {
    const int r = i >> 3, c = i & 7;
    if (c / 2 <= (r & 63) / 16) cp_async16(dst + (r * kCkRow + c * 8) * 2, src + r * kChunk + c * 8, 16);
  }
}

// The warp's 16 x 64 transposed results to rows of `tile` (its own 16 columns), then to `dst` in 32-byte pieces.
__device__ __forceinline__ void store_out(const float (&o)[8][4], __nv_bfloat16* tile, int stride, __nv_bfloat16* dst,
                                          int64_t dst_stride, int nt, int cols, int lane) {
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  __syncwarp();
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) tile[(n * 8 + c2 + (e & 1)) * stride + g + (e >> 1) * 8] = __float2bfloat16_rn(o[n][e]);
  __syncwarp();
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = i * 16 + (lane >> 1), c = (lane & 1) * 8;
    if (r < nt && c < cols) *reinterpret_cast<uint4*>(dst + r * dst_stride + c) = *reinterpret_cast<const uint4*>(tile + r * stride + c);
  }
}

constexpr int kChunkThreads = 256;       // of the second kernel; warps without columns of their own only fetch tiles
// Value columns per CTA of the second kernel: all of them, or fewer when there are few (sequence, head) pairs.
inline int chunk_columns(int64_t pairs, int V) {
  int pb = std::min(128, (V + 15) / 16 * 16);
  while (pb > 32 && pairs * ((V + pb - 1) / pb) * 2 <= kNumSMs) pb = (pb / 2 + 15) / 16 * 16;
  return pb;
}

template <typename F> int chunk_dispatch(int K, F&& f) {
  if (K <= 32) return f(std::integral_constant<int, 32>{});
  if (K <= 64) return f(std::integral_constant<int, 64>{});
  if (K <= 96) return f(std::integral_constant<int, 96>{});
  return f(std::integral_constant<int, 128>{});
}
inline bool chunk_takes(int K, int V) { return K > 0 && V > 0 && K % 8 == 0 && V % 8 == 0 && K <= 128; }
inline int chunk_padded(int K) { return K <= 32 ? 32 : K <= 64 ? 64 : K <= 96 ? 96 : 128; }

}  // namespace mv
