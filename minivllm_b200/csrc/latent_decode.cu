// Decode attention over the paged latent cache, absorbed form, bf16: one query row per sequence and head, all heads
// of a sequence share the cached rows [c | rotated key part], and the value is the c part of the same row, so a row
// that is in shared memory serves the score and the sum.
//
// The batch's 32-key tiles form one stream that is cut into equal ranges, one per worker (the grid depends on shapes
// only; the cut on the device-side lengths).  A CTA holds two workers of 256 threads that share nothing but the SM: one
// computes a softmax while the other keeps the tensor pipe busy.  A range may end or begin inside a sequence: those
// pieces go to the workspace as (m, l, unnormalised sum) and latent_combine_kernel joins them; whole sequences are
// written directly.  Tiles arrive by TMA as 64-column boxes with the 128-byte swizzle (no bank conflicts under
// ldmatrix), two in flight across sequence borders.  16 heads per worker are the 16 rows of m16n8k16 MMAs; eight warps:
// for the scores two key groups times four quarters of the row, the query fragments of its quarter in registers; two
// softmax rows per warp, fp32; for the sum, 16-column units of c (with at most 128 keys the weights enter as two bf16
// terms, value and rounding residue).  The products run without branches, so that loads and
// MMAs of several steps overlap: a step or unit that the sizes do not have works on zeros (queries) or on keys that are
// there, and its result is not stored.  The learned sink joins the denominator when a sequence is finished.
//
// HBM-bound: bytes = sum(ctx) * (rank + rot_dim) * 2.
#include <algorithm>
#include "mma.cuh"
#include "tcgen05.cuh"
#include "tmap.cuh"
#include "vec.cuh"

namespace mv {

constexpr int kLdWorkers = 2;             // per CTA
constexpr int kLdThreads = 256, kLdWarps = 8;   // per worker
constexpr int kLdKeys = 32, kLdHeads = 16, kLdQuarters = 4;
constexpr int kLdMaxSeqs = 1024, kLdMaxRank = 512, kLdMaxRow = 576;
constexpr int kLdUnits = kLdMaxRank / 16 / kLdWarps;   // 16-column units of the sum per warp
constexpr int kLdBox = kLdKeys * 128;       // bytes of a box of 32 keys, 64 columns
constexpr int kLdAhead = 128;                // tiles whose cache rows are known ahead
constexpr int kLdFewKeys = 128;
constexpr int kLdQPieces = (kLdHeads * kLdMaxRow / 8 + kLdThreads - 1) / kLdThreads;   // 16-byte pieces of the queries per thread
constexpr int kLdSStride = kLdKeys + 4;    // floats per score row
constexpr int kLdPStride = kLdKeys + 8;    // bf16 per weight row

struct LdParams {
  __nv_bfloat16* out; int64_t out_stride, out_head_stride;
  const __nv_bfloat16* q_lat; int64_t q_lat_stride, q_lat_head_stride;
  const __nv_bfloat16* q_rot; int64_t q_rot_stride, q_rot_head_stride;
  int box_rows;                  // rows of one TMA box: 32, or the block size when that is smaller
  const int32_t* tables; int64_t bt_stride; int max_blocks, block_size; int64_t num_blocks;
  const int64_t* positions;      // keys of sequence b: positions[b] + 1
  const int32_t* active;         // null, or per sequence < 0: a padding row without keys
  const __nv_bfloat16* sink;
  int batch, heads, rank, rot_dim;
  float scale_log2;
  int* error_word;
  float* ws;                     // [head tile][cta][2] pieces of {m[16], l[16], acc[16][rank]} (cta: worker)
};

__host__ __device__ inline int64_t ld_piece_floats(int rank) { return 2 * kLdHeads + static_cast<int64_t>(kLdHeads) * rank; }
// shared memory of a worker behind its tile buffers: queries, scores, weights
__host__ __device__ inline int ld_rest_bytes(int row_bytes) {
  return kLdHeads * row_bytes + kLdQuarters * kLdHeads * kLdSStride * 4 + 2 * kLdHeads * kLdPStride * 2;
}
__device__ __forceinline__ int ld_tiles(const LdParams& p, int b) {
  if (p.active && p.active[b] < 0) return 0;
  const int64_t n = min(p.positions[b] + 1, static_cast<int64_t>(p.max_blocks) * p.block_size);
  return static_cast<int>((n + kLdKeys - 1) / kLdKeys);
}
// s_keys[b] = keys of sequence b (kKeys), s_start[b] = tiles before sequence b, s_start[batch] = all
template <bool kKeys>
__device__ __forceinline__ void ld_prefix(const LdParams& p, int* s_start, int* s_keys) {
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    int carry = 0;
    for (int base = 0; base < p.batch; base += 32) {
      const int b = base + lane, n = b < p.batch ? ld_tiles(p, b) : 0;
      int incl = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += v;
      }
      if (b < p.batch) s_start[b] = carry + incl - n;
      if (kKeys && b < p.batch) s_keys[b] = n ? static_cast<int>(min(p.positions[b] + 1, static_cast<int64_t>(p.max_blocks) * p.block_size)) : 0;
      carry += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (lane == 0) s_start[p.batch] = carry;
  }
  __syncthreads();
}
__device__ __forceinline__ int ld_cut(int total, int c, int ctas) { return static_cast<int>(static_cast<int64_t>(total) * c / ctas); }

// kSteps: 16-column steps of a quarter of a row that the query fragments have registers for.  kRank, kRow: sizes known at
// compile time (0: any), which leaves the tile loop without spilled addresses.
template <int kSteps, int kRank = 0, int kRow = 0>
__global__ void __launch_bounds__(kLdWorkers * kLdThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmap, const LdParams p) {
  extern __shared__ unsigned char raw[];
  __shared__ int s_start[kLdMaxSeqs + 1], s_keys[kLdMaxSeqs];
  __shared__ float s_ml[kLdWorkers][3][kLdHeads];
  __shared__ __align__(8) uint64_t s_bar[kLdWorkers][2];
  __shared__ int s_abort, s_rows[kLdWorkers][kLdAhead][4];
  const int wk = threadIdx.x / kLdThreads, tid = threadIdx.x % kLdThreads, warp = tid >> 5, lane = tid & 31;
  const int rank = kRank ? kRank : p.rank, R = kRow ? kRow : p.rank + p.rot_dim, row_bytes = R * 2 + 16;
  const int boxes = (R + 63) / 64;
  const uint32_t base = (smem_u32(raw) + 1023u) & ~1023u;
  const uint32_t kv_s = base + wk * 2 * boxes * kLdBox;      // [2][box][32][128B], swizzled
  unsigned char* rest = raw + (base - smem_u32(raw)) + kLdWorkers * 2 * boxes * kLdBox + wk * ld_rest_bytes(row_bytes);
  unsigned char* sq = rest;                                                              // [16][row_bytes]
  float* ss = reinterpret_cast<float*>(sq + kLdHeads * row_bytes);                       // [quarter][16][kLdSStride]
  __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(ss + kLdQuarters * kLdHeads * kLdSStride);  // [2 terms][16][kLdPStride]
  float *s_m = s_ml[wk][0], *s_l = s_ml[wk][1], *s_c = s_ml[wk][2];
  int (*s_row)[4] = s_rows[wk];
  const uint32_t q_s = smem_u32(sq), p_s = smem_u32(sp), bar0 = smem_u32(s_bar[wk]);
  const int h0 = blockIdx.y * kLdHeads, nh = min(kLdHeads, p.heads - h0);
  auto sync = [&] { asm volatile("bar.sync %0, %1;" ::"r"(1 + wk), "n"(kLdThreads) : "memory"); };
  if (threadIdx.x == 0) {
    s_abort = *reinterpret_cast<volatile int*>(p.error_word) != 0;    // an earlier wait ran out: do nothing
    for (int i = 0; i < 2 * kLdWorkers; ++i) tc::mbar_init(smem_u32(&s_bar[0][0]) + 8 * i, 1);
    tc::mbar_fence_init();
  }
  ld_prefix<true>(p, s_start, s_keys);
  const int total = s_abort ? 0 : s_start[p.batch], ctas = gridDim.x * kLdWorkers, c = blockIdx.x * kLdWorkers + wk;
  const int g0 = ld_cut(total, c, ctas), g1 = ld_cut(total, c + 1, ctas);
  if (g0 >= g1) return;         // the whole worker; from here on it only meets its own barrier
  // Cache rows of the tiles ahead, looked up by all threads for 64 tiles at a time (a lookup in the block table takes
  // as long as a tile's scores).  A missing block is a row outside the tensor and reads as zeros.
  const int groups = kLdKeys / p.box_rows;        // boxes of rows per tile
  auto find = [&](int g) {      // the sequence of tile g: the last b with s_start[b] <= g
    int lo = 0, hi = p.batch - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (s_start[mid] <= g) lo = mid; else hi = mid - 1;
    }
    return lo;
  };
  auto look = [&](int first, int tiles) {
    for (int i = tid; i < tiles * groups; i += kLdThreads) {
      const int g = first + i / groups, r = i % groups;
      if (g >= g1) break;
      const int sb = find(g), pos = (g - s_start[sb]) * kLdKeys + r * p.box_rows, blk = pos / p.block_size;
      const int32_t phys = pos < s_keys[sb] ? p.tables[static_cast<int64_t>(sb) * p.bt_stride + blk] : -1;
      s_row[(g - g0) % kLdAhead][r] = phys >= 0 && phys < p.num_blocks ? phys * p.block_size + (pos - blk * p.block_size)
                                                                      : static_cast<int>(p.num_blocks) * p.block_size;
    }
  };
  // Every warp copies its boxes of a tile: nine copies issued by one thread would take longer than the tile's products.
  auto load = [&](int g, int buf) {
    if (g >= g1) return;
    if (tid == 0) tc::mbar_expect_tx(bar0 + 8 * buf, boxes * kLdBox);
    __syncwarp();
    for (int x = warp; x < boxes; x += kLdWarps)
      for (int r = 0; r < groups; ++r)
        tc::tma_load_3d_elected(kv_s + (buf * boxes + x) * kLdBox + r * p.box_rows * 128, &tmap, x * 64,
                                s_row[(g - g0) % kLdAhead][r], 0, bar0 + 8 * buf);
  };
  // A sequence's queries: all pieces requested at once, and before they are needed.
  auto load_q = [&](int b) {
    int t = tid, chunks = R / 8;
    asm volatile("" : "+r"(t), "+r"(chunks));     // computed here and not kept in registers across the tiles
    uint4 raw[kLdQPieces];
#pragma unroll
    for (int k = 0; k < kLdQPieces; ++k) {
      const int i = t + k * kLdThreads, h = i / chunks, col = (i - h * chunks) * 8;
      raw[k] = make_uint4(0, 0, 0, 0);
      if (h < nh)
        raw[k] = *reinterpret_cast<const uint4*>(col < rank ? p.q_lat + b * p.q_lat_stride + (h0 + h) * p.q_lat_head_stride + col
                                                              : p.q_rot + b * p.q_rot_stride + (h0 + h) * p.q_rot_head_stride + col - rank);
    }
#pragma unroll
    for (int k = 0; k < kLdQPieces; ++k) {
      const int i = t + k * kLdThreads, h = i / chunks, col = (i - h * chunks) * 8;
      if (h < kLdHeads) *reinterpret_cast<uint4*>(sq + h * row_bytes + col * 2) = raw[k];
    }
  };
  int b = find(g0), first_g = g0;
  look(g0, 2);
  sync();
  load(g0, 0);
  load(g0 + 1, 1);
  look(g0 + 2, kLdAhead - 2);      // while the first tiles are on their way
  load_q(b);
  sync();

  const int steps = R / 16, per = (steps + kLdQuarters - 1) / kLdQuarters;
  const int kt = warp & 1, quarter = warp >> 1;       // score role: 16 keys, a quarter of the row
  const int k_first = quarter * per;
  const int units = rank / 16;
  uint32_t qf[kSteps][4];
  float acc[kLdUnits][8];
  float m_row[2], l_lane[2];     // softmax rows of this warp: running maximum, this lane's part of the sum
  bool fresh = true;
  int nkeys = 0;
  for (int g = g0; g < g1; ++g) {
    const int buf = (g - g0) & 1;
    while (g >= s_start[b + 1]) ++b;
    if (fresh) {
      first_g = g;
      nkeys = s_keys[b];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        m_row[i] = -INFINITY;
        l_lane[i] = 0.f;
      }
#pragma unroll
      for (int i = 0; i < kLdUnits; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;
      const uint32_t qa = q_s + ((lane & 7) + ((lane >> 3) & 1) * 8) * row_bytes + (lane >> 4) * 16 + k_first * 32;
#pragma unroll
      for (int k = 0; k < kSteps; ++k) {
        uint32_t a[4] = {0, 0, 0, 0};
        if (k < per && k_first + k < steps) ldmatrix_x4(a, qa + k * 32);
#pragma unroll
        for (int j = 0; j < 4; ++j) qf[k][j] = a[j];
      }
      fresh = false;
    }
    tc::mbar_wait(bar0 + 8 * buf, ((g - g0) >> 1) & 1, &s_abort, p.error_word, 0x50);   // out of time: run on, the host learns of it
    const uint32_t kb = kv_s + buf * boxes * kLdBox;
    {  // scores of 16 keys over a quarter of the row
      float d[2][4] = {};
      const uint32_t ka = kb + (kt * 16 + (lane & 7) + (lane >> 4) * 8) * 128;
      const int half = (lane >> 3) & 1, sw = lane & 7;
#pragma unroll
      for (int k = 0; k < kSteps; ++k) {
        uint32_t kf[4];
        const int st = min(k_first + k, steps - 1);
        ldmatrix_x4(kf, ka + (st >> 2) * kLdBox + ((((st & 3) * 2 + half) ^ sw) << 4));
        Mma16816<__nv_bfloat16>::run(d[0], qf[k], kf[0], kf[1]);
        Mma16816<__nv_bfloat16>::run(d[1], qf[k], kf[2], kf[3]);
      }
      float* o = ss + (quarter * kLdHeads + (lane >> 2)) * kLdSStride + kt * 16 + (lane & 3) * 2;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        *reinterpret_cast<float2*>(o + j * 8) = make_float2(d[j][0], d[j][1]);
        *reinterpret_cast<float2*>(o + j * 8 + 8 * kLdSStride) = make_float2(d[j][2], d[j][3]);
      }
    }
    sync();
    {  // two rows per warp, a key per lane
      const bool on = lane < nkeys - (g - s_start[b]) * kLdKeys;
      float v[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float* r = ss + (warp * 2 + i) * kLdSStride + lane;
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < kLdQuarters; ++k) s += r[k * kLdHeads * kLdSStride];
        v[i] = on ? s * p.scale_log2 : -INFINITY;
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int h = warp * 2 + i;
        float mx;
        asm("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(mx) : "f"(v[i]));
        const float m_new = fmaxf(m_row[i], mx), corr = fast_exp2(m_row[i] - m_new);
        const float w = fast_exp2(v[i] - m_new);      // key 0 of a tile is always visible
        l_lane[i] = fmaf(l_lane[i], corr, w);
        m_row[i] = m_new;
        const __nv_bfloat16 hi = __float2bfloat16_rn(w);
        sp[h * kLdPStride + lane] = hi;
        sp[(kLdHeads + h) * kLdPStride + lane] = __float2bfloat16_rn(w - __bfloat162float(hi));
        if (lane == 0) s_c[h] = corr;
      }
    }
    sync();
    {  // weighted sum: this warp's 16-column units, all keys
      const float c0 = s_c[lane >> 2], c1 = s_c[(lane >> 2) + 8];
#pragma unroll
      for (int i = 0; i < kLdUnits; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] *= (j & 2) ? c1 : c0;
      const uint32_t pa = p_s + (((lane & 7) + ((lane >> 3) & 1) * 8) * kLdPStride + (lane >> 4) * 8) * 2;
      const uint32_t vo = ((lane & 7) + ((lane >> 3) & 1) * 8) * 128 + ((((warp & 3) * 2 + (lane >> 4)) ^ (lane & 7)) * 16);
      auto add = [&](uint32_t weights) {
#pragma unroll
        for (int k = 0; k < kLdKeys; k += 16) {
          uint32_t w[4];
          ldmatrix_x4(w, weights + k * 2);
#pragma unroll
          for (int i = 0; i < kLdUnits; ++i) {
            uint32_t v[4];
            ldmatrix_x4_trans(v, kb + min((warp >> 2) + i * (kLdWarps / 4), boxes - 1) * kLdBox + vo + k * 128);
            Mma16816<__nv_bfloat16>::run(*reinterpret_cast<float (*)[4]>(&acc[i][0]), w, v[0], v[1]);
            Mma16816<__nv_bfloat16>::run(*reinterpret_cast<float (*)[4]>(&acc[i][4]), w, v[2], v[3]);
          }
        }
      };
      add(pa);
      // with few keys the rounding of the weights does not average out: their residues are added too
      if (nkeys <= kLdFewKeys) add(pa + kLdHeads * kLdPStride * 2);
    }
    sync();           // the buffer and the weights are free again
    load(g + 2, buf);
    if ((g - g0) % (kLdAhead / 2) == kLdAhead / 2 - 1) look(g + 1 + kLdAhead / 2, kLdAhead / 2);   // over rows already used
    const bool last = g + 1 == s_start[b + 1];
    if (last || g + 1 == g1) {
      const bool whole = last && first_g == s_start[b];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float l_row = warp_sum(l_lane[i]);
        if (lane == 0) { s_m[warp * 2 + i] = m_row[i]; s_l[warp * 2 + i] = l_row; }
      }
      sync();
      const int r = lane >> 2, col = (lane & 3) * 2;
      float* piece = p.ws + ((static_cast<int64_t>(blockIdx.y) * ctas + c) * 2 + (first_g == g0 ? 0 : 1)) * ld_piece_floats(rank);
      if (!whole && tid < kLdHeads) { piece[tid] = s_m[tid]; piece[kLdHeads + tid] = s_l[tid]; }
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int h = r + hf * 8;
        float inv = 1.f;
        if (whole) {
          float m = s_m[h], l = s_l[h], f = 1.f;
          if (p.sink && h < nh) {
            const float sk = __bfloat162float(p.sink[h0 + h]) * 1.4426950408889634f, mm = fmaxf(m, sk);
            f = exp2f(m - mm);
            l = l * f + exp2f(sk - mm);
          }
          inv = l > 0.f ? f / l : 0.f;
        }
#pragma unroll
        for (int i = 0; i < kLdUnits; ++i)
          if (warp + i * kLdWarps < units) {
#pragma unroll
            for (int t = 0; t < 2; ++t) {
              const int at = (warp + i * kLdWarps) * 16 + t * 8 + col;
              const float x = acc[i][t * 4 + hf * 2], y = acc[i][t * 4 + hf * 2 + 1];
              if (!whole) *reinterpret_cast<float2*>(piece + 2 * kLdHeads + h * rank + at) = make_float2(x, y);
              else if (h < nh)
                *reinterpret_cast<__nv_bfloat162*>(p.out + b * p.out_stride + (h0 + h) * p.out_head_stride + at) =
                    __floats2bfloat162_rn(x * inv, y * inv);
            }
          }
      }
      if (g + 1 < g1) {          // the next sequence's queries: every warp has its fragments of this one's
        int nb = b + 1;
        while (g + 1 >= s_start[nb + 1]) ++nb;
        load_q(nb);
      }
      sync();         // queries of the next sequence are there, s_m and s_l are free
      fresh = true;
    }
  }
  if (*reinterpret_cast<volatile int*>(&s_abort) && tid == 0)      // copies in flight must land before the shared memory goes away
    for (int g = max(g0, g1 - 2); g < g1; ++g) tc::mbar_wait_timed(bar0 + 8 * ((g - g0) & 1), ((g - g0) >> 1) & 1);
  sync();
}

// One CTA per (sequence, head): joins the pieces of a sequence that several workers had a part of.  Sequences without keys
// (padding rows) get zeros.
__global__ void __launch_bounds__(128) latent_combine_kernel(const LdParams p, int ctas) {
  __shared__ int s_start[kLdMaxSeqs + 1];
  __shared__ float s_w[kLdWorkers * kNumSMs + 1];
  __shared__ int s_piece[kLdWorkers * kNumSMs + 1];
  __shared__ float s_inv;
  __shared__ int s_n;
  ld_prefix<false>(p, s_start, nullptr);
  const int b = blockIdx.x, h = blockIdx.y, total = s_start[p.batch], t0 = s_start[b], t1 = s_start[b + 1];
  __nv_bfloat16* o = p.out + b * p.out_stride + h * p.out_head_stride;
  if (t0 == t1) {
    for (int d = threadIdx.x; d < p.rank; d += 128) o[d] = __float2bfloat16_rn(0.f);
    return;
  }
  const int64_t pf = ld_piece_floats(p.rank);
  const float* base = p.ws + static_cast<int64_t>(h / kLdHeads) * ctas * 2 * pf;
  const int r = h % kLdHeads;
  if (threadIdx.x < 32) {      // a warp collects the pieces: workers whose range meets [t0, t1), in order
    const int lane = threadIdx.x;
    int guess = static_cast<int>(static_cast<int64_t>(t0) * ctas / total) - 1;
    if (guess < 0) guess = 0;
    int n = 0;
    for (int c0 = guess; c0 < ctas; c0 += 32) {
      const int c = c0 + lane;
      const int lo = c < ctas ? ld_cut(total, c, ctas) : total, hi = c < ctas ? ld_cut(total, c + 1, ctas) : total;
      const bool mine = lo < hi && lo < t1 && hi > t0;
      const uint32_t mask = __ballot_sync(0xffffffffu, mine);
      if (mine) s_piece[n + __popc(mask & ((1u << lane) - 1))] = c * 2 + (lo < t0 ? 1 : 0);
      n += __popc(mask);
      if (__shfl_sync(0xffffffffu, lo, 31) >= t1) break;
    }
    __syncwarp();
    const float sk = p.sink ? __bfloat162float(p.sink[h]) * 1.4426950408889634f : -INFINITY;
    float m = sk;
    for (int i = lane; i < n; i += 32) m = fmaxf(m, base[s_piece[i] * pf + r]);
#pragma unroll
    for (int k = 16; k; k >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, k));
    float l = 0.f;
    for (int i = lane; i < n; i += 32) {
      const float w = exp2f(base[s_piece[i] * pf + r] - m);
      s_w[i] = w;
      l = fmaf(base[s_piece[i] * pf + kLdHeads + r], w, l);
    }
    l = warp_sum(l) + (p.sink ? exp2f(sk - m) : 0.f);
    if (lane == 0) {
      s_inv = l > 0.f ? 1.f / l : 0.f;
      s_n = n;
    }
  }
  __syncthreads();
  const int n = s_n;
  if (n < 2) return;           // one worker had all of it and wrote it
  const float inv = s_inv;
  for (int d = threadIdx.x * 4; d < p.rank; d += 512) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int i = 0; i < n; ++i) {
      const float4 v = *reinterpret_cast<const float4*>(base + s_piece[i] * pf + 2 * kLdHeads + r * p.rank + d);
      const float w = s_w[i];
      a.x = fmaf(v.x, w, a.x); a.y = fmaf(v.y, w, a.y); a.z = fmaf(v.z, w, a.z); a.w = fmaf(v.w, w, a.w);
    }
    *reinterpret_cast<__nv_bfloat162*>(o + d) = __floats2bfloat162_rn(a.x * inv, a.y * inv);
    *reinterpret_cast<__nv_bfloat162*>(o + d + 2) = __floats2bfloat162_rn(a.z * inv, a.w * inv);
  }
}

static bool ld_takes(int batch, int rank, int rot_dim) {
  return batch <= kLdMaxSeqs && rank % 16 == 0 && rank <= kLdMaxRank && (rank + rot_dim) % 32 == 0 && rank + rot_dim <= kLdMaxRow;
}
static int ld_ctas(int heads) { return std::max(1, kNumSMs / ((heads + kLdHeads - 1) / kLdHeads)); }

}  // namespace mv

extern "C" int64_t mv_latent_decode_workspace_bytes(int batch, int heads, int rank, int rot_dim) {
  using namespace mv;
  if (batch < 0 || heads <= 0 || rank <= 0 || rot_dim < 0 || !ld_takes(batch, rank, rot_dim)) return -1;
  return static_cast<int64_t>((heads + kLdHeads - 1) / kLdHeads) * ld_ctas(heads) * kLdWorkers * 2 * ld_piece_floats(rank) * 4;
}

extern "C" int mv_latent_decode(void* out, int64_t out_stride, int64_t out_head_stride, const void* q_lat,
                                int64_t q_lat_stride, int64_t q_lat_head_stride, const void* q_rot,
                                int64_t q_rot_stride, int64_t q_rot_head_stride, const void* cache,
                                const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size,
                                int64_t num_blocks, const int64_t* positions, const int32_t* active, const void* sink,
                                int batch, int heads, int rank, int rot_dim, float scale, void* workspace,
                                int64_t workspace_bytes, int* error_word, void* stream) {
  using namespace mv;
  if (batch < 0 || heads <= 0 || block_size <= 0 || max_blocks < 0) return fail(MV_ERR_SHAPE, "latent_decode: batch %d heads %d", batch, heads);
  if (!ld_takes(batch, rank, rot_dim)) return fail(MV_ERR_LIMIT, "latent_decode: batch %d rank %d rot_dim %d", batch, rank, rot_dim);
  if (batch == 0) return MV_OK;
  if (!out || !q_lat || (rot_dim && !q_rot) || !cache || !block_tables || !positions || !workspace || !error_word)
    return fail(MV_ERR_NULL, "latent_decode: null pointer");
  if (workspace_bytes < mv_latent_decode_workspace_bytes(batch, heads, rank, rot_dim)) return fail(MV_ERR_WORKSPACE, "latent_decode: workspace");
  if (!vec8_ok(q_lat, q_lat_stride, 2) || q_lat_head_stride % 8 ||
      (rot_dim && (!vec8_ok(q_rot, q_rot_stride, 2) || q_rot_head_stride % 8)) ||
      !aligned16(cache) || !vec8_ok(out, out_stride, 2) || out_head_stride % 8 || !aligned16(workspace))
    return fail(MV_ERR_ALIGN, "latent_decode: rows must start on 16-byte boundaries");
  LdParams p{static_cast<__nv_bfloat16*>(out), out_stride, out_head_stride, static_cast<const __nv_bfloat16*>(q_lat),
             q_lat_stride, q_lat_head_stride, static_cast<const __nv_bfloat16*>(q_rot), q_rot_stride, q_rot_head_stride,
             block_size % kLdKeys == 0 ? kLdKeys : block_size, block_tables, bt_stride, max_blocks, block_size, num_blocks,
             positions, active, static_cast<const __nv_bfloat16*>(sink), batch, heads, rank, rot_dim,
             scale * 1.4426950408889634f, error_word, static_cast<float*>(workspace)};
  if (block_size % kLdKeys && (kLdKeys % block_size || block_size < 8))
    return fail(MV_ERR_SHAPE, "latent_decode: block_size %d", block_size);
  if (num_blocks * block_size > 0x7fffff00LL) return fail(MV_ERR_LIMIT, "latent_decode: cache of %lld rows", static_cast<long long>(num_blocks * block_size));
  CUtensorMap tm;
  const int64_t cache_rows = num_blocks * block_size, R = rank + rot_dim;
  const int rct = make_tmap_bf16(&tm, cache, R, cache_rows, 1, R, cache_rows * R, p.box_rows, 1, "latent_decode");
  if (rct) return rct;
  const int row_bytes = (rank + rot_dim) * 2 + 16;
  const size_t smem = 1024 + static_cast<size_t>(kLdWorkers) * (2 * ((rank + rot_dim + 63) / 64) * kLdBox + ld_rest_bytes(row_bytes));
  const int ctas = ld_ctas(heads);
  auto st = static_cast<cudaStream_t>(stream);
  auto go = [&](auto kernel) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "latent_decode: %s", cudaGetErrorString(e));
    kernel<<<dim3(ctas, (heads + kLdHeads - 1) / kLdHeads), kLdWorkers * kLdThreads, smem, st>>>(tm, p);
    return check_launch("latent_decode");
  };
  const int rc = rank == 512 && rot_dim == 64 ? go(latent_decode_kernel<9, 512, 576>) : rank + rot_dim <= 320 ? go(latent_decode_kernel<5>) : go(latent_decode_kernel<9>);
  if (rc) return rc;
  latent_combine_kernel<<<dim3(batch, heads), 128, 0, st>>>(p, ctas * kLdWorkers);
  return check_launch("latent_decode");
}
