// Grouped-query attention whose softmax weights are mixed across the heads ("talking heads"), with capped scores and a bias that
// grows with the logarithm of the distance, over a paged cache of rows [keys of all KV heads | values of all KV heads]:
//   s = cap tanh(scale (q . k) / cap) - r1[h] ln(1 + r2[h] distance),  w = softmax(s),  w'_h = sum_g talk[h, g] w_g
//   out_h = sum_j w'_h(j) v_j of h's own value head
// A capped score needs no running maximum: e^s is formed as it is, for caps up to kTalkCap.
//
// One token per sequence (bf16, HBM-bound on the cache rows, each read once):
//   talk_scores_kernel  e^s of every head and key to scratch (fp32), sums per head and piece
//   talk_values_kernel  per value head: the mixture of all heads' weights, divided by their sums, times the values; both
//                       products on mma.sync, weights and mixture as value and rounding residue
//   talk_join_kernel    sums the pieces
// head_mix_kernel       the mixture for results [token][weight head][value head] (prompts: talk_prefill.cu; any sizes:
//                       window_attention.cu): out_h = sum_g talk[h, g] a[g, value head of h]
#include <algorithm>
#include <type_traits>
#include "mma.cuh"
#include "talk.cuh"
#include "vec.cuh"

namespace mv {

constexpr int kTkWarps = 4, kTkThreads = 32 * kTkWarps, kTkStages = 3, kTkTile = 16;
constexpr int kTkRow = 20;                     // floats between the heads of a tile of weights in shared memory

struct TalkParams {
  __nv_bfloat16* out; int64_t out_stride;      // (batch, heads * vdim)
  const __nv_bfloat16* q; int64_t q_stride;
  const __nv_bfloat16* cache;
  const int32_t* tables; int64_t bt_stride; int max_blocks, block_size; int64_t num_blocks;
  const int64_t* positions;
  const float *r1, *r2, *talk;                 // (heads), (heads), (heads, heads)
  int heads, kv_heads, dim, vdim;
  float scale, cap, out_scale;
  int splits, steps; int64_t keys;             // pieces; k-steps of 16 weight heads; padded keys per head in `weights`
  float *weights, *sums, *part;                // (batch, heads, keys), (batch, heads, splits), (batch, splits, heads, vdim)
};

// Where the piece of a sequence lies that this CTA works on, in tiles of 16 keys.
struct TalkPiece {
  int begin, end, tiles;
  __device__ __forceinline__ TalkPiece(const TalkParams& p, int64_t pos, int split) {
    const int nk = static_cast<int>(min(pos + 1, static_cast<int64_t>(p.max_blocks) * p.block_size));
    const int len = ((nk + p.splits - 1) / p.splits + kTkTile - 1) / kTkTile * kTkTile;
    begin = split * len;
    end = min(begin + len, nk);
    tiles = end > begin ? (end - begin + kTkTile - 1) / kTkTile : 0;
  }
};
// Offset of key `at`'s row in the cache, in rows; -1 without one.
__device__ __forceinline__ int64_t talk_row(const TalkParams& p, const int32_t* table, int at, int end) {
  const int blk = at / p.block_size;
  if (at >= end || blk >= p.max_blocks) return -1;
  const int32_t phys = __ldg(table + blk);
  return phys >= 0 && phys < p.num_blocks ? static_cast<int64_t>(phys) * p.block_size + (at - blk * p.block_size) : -1;
}
// cp.async of 16 rows of C 16-byte pieces (`real` of them in memory), swizzled; lane l knows row l & 15 (in elements, -1: zeros).
template <int C> __device__ __forceinline__ void talk_fetch(uint32_t dst, const __nv_bfloat16* base, int64_t at, int real, int lane) {
#pragma unroll
  for (int c0 = 0; c0 < kTkTile * C; c0 += 32) {
    const int r = (c0 + lane) / C, c = (c0 + lane) % C;
    const int64_t src = __shfl_sync(0xffffffffu, at, r);
    const bool ok = src >= 0 && c < real;
    cp_async16(dst + r * (C * 16) + ((c ^ (r & 7)) << 4), ok ? base + src + c * 8 : base, ok ? 16 : 0);
  }
}

template <int KD>
__global__ void __launch_bounds__(kTkThreads) talk_scores_kernel(const TalkParams p) {
  using Mma = Mma16816<__nv_bfloat16>;
  constexpr int KSTEPS = KD / 16, kStage = kTkTile * KD * 2;
  extern __shared__ __align__(128) unsigned char smem[];
  __shared__ uint32_t s_live[kTkWarps][kTkStages];
  __shared__ float s_sum[kTkWarps][16];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int group = p.heads / p.kv_heads, mtiles = (group + 15) / 16;
  const int kv = blockIdx.y / mtiles, mt = blockIdx.y - kv * mtiles, b = blockIdx.z;
  const int rows = min(16, group - mt * 16), h0 = kv * group + mt * 16;
  const int pos = static_cast<int>(p.positions[b]);
  const TalkPiece piece(p, pos, blockIdx.x);
  const int mine = piece.tiles > warp ? (piece.tiles - warp + kTkWarps - 1) / kTkWarps : 0;
  const int32_t* table = p.tables + static_cast<int64_t>(b) * p.bt_stride;
  const int64_t row = static_cast<int64_t>(p.kv_heads) * (p.dim + p.vdim);
  const uint32_t ring = smem_u32(smem) + warp * kTkStages * kStage;
  auto issue = [&](int i) {
    if (i < mine) {
      const int64_t at = talk_row(p, table, piece.begin + (i * kTkWarps + warp) * kTkTile + (lane & 15), piece.end);
      const uint32_t live = __ballot_sync(0xffffffffu, at >= 0) & 0xffffu;
      if (lane == 0) s_live[warp][i % kTkStages] = live;
      talk_fetch<KD / 8>(ring + i % kTkStages * kStage, p.cache + kv * p.dim, at < 0 ? -1 : at * row, p.dim / 8, lane);
    }
    cp_async_commit();
  };
#pragma unroll
  for (int i = 0; i < kTkStages - 1; ++i) issue(i);
  uint32_t qa[KSTEPS][4];
  {
    const __nv_bfloat16* qb = p.q + b * p.q_stride + static_cast<int64_t>(h0) * p.dim;
    const uint32_t* q0 = reinterpret_cast<const uint32_t*>(qb + static_cast<int64_t>(g) * p.dim);
    const uint32_t* q1 = reinterpret_cast<const uint32_t*>(qb + static_cast<int64_t>(g + 8) * p.dim);
    const bool v0 = g < rows, v1 = g + 8 < rows;
    const int half = p.dim / 2;
#pragma unroll
    for (int ks = 0; ks < KSTEPS; ++ks) {
      const int c = ks * 8 + t;
      qa[ks][0] = v0 && c < half ? __ldg(q0 + c) : 0u;
      qa[ks][1] = v1 && c < half ? __ldg(q1 + c) : 0u;
      qa[ks][2] = v0 && c + 4 < half ? __ldg(q0 + c + 4) : 0u;
      qa[ks][3] = v1 && c + 4 < half ? __ldg(q1 + c + 4) : 0u;
    }
  }
  const TalkScore score(p.scale, p.cap);
  const int ha = h0 + min(g, rows - 1), hb = h0 + min(g + 8, rows - 1);
  const float r1[2] = {p.r1[ha], p.r1[hb]}, r2[2] = {p.r2[ha], p.r2[hb]};
  float* out[2] = {p.weights + (static_cast<int64_t>(b) * p.heads + ha) * p.keys, p.weights + (static_cast<int64_t>(b) * p.heads + hb) * p.keys};
  float sum[2] = {0.f, 0.f};
  for (int i = 0; i < mine; ++i) {
    cp_async_wait<kTkStages - 2>();
    __syncwarp();
    const int k0 = piece.begin + (i * kTkWarps + warp) * kTkTile;
    const uint32_t kd = ring + i % kTkStages * kStage, live = s_live[warp][i % kTkStages];
    float s[2][4] = {};
    const int r = (lane & 7) + ((lane >> 4) << 3), csel = (lane >> 3) & 1;
#pragma unroll
    for (int ks = 0; ks < KSTEPS; ++ks) {
      uint32_t kb[4];
      ldmatrix_x4(kb, kd + r * (KD * 2) + (((2 * ks + csel) ^ (r & 7)) << 4));
      Mma::run(s[0], qa[ks], kb[0], kb[1]);
      Mma::run(s[1], qa[ks], kb[2], kb[3]);
    }
    issue(i + kTkStages - 1);
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float2 w;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int col = n * 8 + 2 * t + e;
          const float v = (live >> col) & 1u ? score.weight(s[n][2 * half + e], score.bias(r1[half], r2[half], pos - k0 - col)) : 0.f;
          (e ? w.y : w.x) = v;
          sum[half] += v;
        }
        if (g + half * 8 < rows) *reinterpret_cast<float2*>(out[half] + k0 + n * 8 + 2 * t) = w;
      }
    __syncwarp();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    sum[half] += __shfl_xor_sync(0xffffffffu, sum[half], 1);
    sum[half] += __shfl_xor_sync(0xffffffffu, sum[half], 2);
    if (t == 0) s_sum[warp][g + half * 8] = sum[half];
  }
  __syncthreads();
  if (tid < rows) {
    float v = 0.f;
    for (int w = 0; w < kTkWarps; ++w) v += s_sum[w][tid];
    p.sums[(static_cast<int64_t>(b) * p.heads + h0 + tid) * p.splits + blockIdx.x] = v;
  }
}

// Bytes of shared memory: the mixture's operand, then the warps' stages (joined in the end).
inline int talk_values_smem(int VD, int steps) {
  const int stage = steps * 16 * kTkRow * 4 + kTkTile * VD * 2, merge = kTkWarps * 16 * (VD + 8) * 4;
  return steps * 1024 + std::max(kTkWarps * kTkStages * stage, merge) + steps * 16 * 4;
}

template <int VD>
__global__ void __launch_bounds__(kTkThreads) talk_values_kernel(const TalkParams p) {
  using Mma = Mma16816<__nv_bfloat16>;
  constexpr int NT = VD / 8, kStride = VD + 8;
  extern __shared__ __align__(128) unsigned char smem[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int group = p.heads / p.kv_heads, mtiles = (group + 15) / 16, H = p.heads;
  const int kv = blockIdx.y / mtiles, mt = blockIdx.y - kv * mtiles, b = blockIdx.z, split = blockIdx.x;
  const int rows = min(16, group - mt * 16), h0 = kv * group + mt * 16;
  const TalkPiece piece(p, p.positions[b], split);
  const int mine = piece.tiles > warp ? (piece.tiles - warp + kTkWarps - 1) / kTkWarps : 0;
  const int32_t* table = p.tables + static_cast<int64_t>(b) * p.bt_stride;
  const int64_t row = static_cast<int64_t>(p.kv_heads) * (p.dim + p.vdim);
  const int w_bytes = p.steps * 16 * kTkRow * 4, stage_bytes = w_bytes + kTkTile * VD * 2;
  uint4* s_mix = reinterpret_cast<uint4*>(smem);                   // [step][hi, lo][lane]
  unsigned char* stages = smem + p.steps * 1024;
  const uint32_t ring = smem_u32(stages) + warp * kTkStages * stage_bytes;
  const float* weights = p.weights + static_cast<int64_t>(b) * H * p.keys;
  auto issue = [&](int i) {
    if (i < mine) {
      const int k0 = piece.begin + (i * kTkWarps + warp) * kTkTile;
      const uint32_t st = ring + i % kTkStages * stage_bytes;
      for (int c = lane; c < p.steps * 64; c += 32) {              // four pieces of every head
        const int h = c >> 2, q = c & 3;
        cp_async16(st + (h * kTkRow + q * 4) * 4, h < H ? weights + h * p.keys + k0 + q * 4 : weights, h < H ? 16 : 0);
      }
      const int64_t at = talk_row(p, table, k0 + (lane & 15), piece.end);
      talk_fetch<VD / 8>(st + w_bytes, p.cache + p.kv_heads * p.dim + kv * p.vdim, at < 0 ? -1 : at * row, p.vdim / 8, lane);
    }
    cp_async_commit();
  };
#pragma unroll
  for (int i = 0; i < kTkStages - 1; ++i) issue(i);
  // the mixture's rows of this value head over the heads' sums, as fragments of an A operand in two terms
  {
    float* s_inv = reinterpret_cast<float*>(stages + std::max(kTkWarps * kTkStages * stage_bytes, kTkWarps * 16 * kStride * 4));
    for (int h = tid; h < p.steps * 16; h += kTkThreads) {
      float l = 0.f;
      if (h < H)
        for (int s = 0; s < p.splits; ++s) l += p.sums[(static_cast<int64_t>(b) * H + h) * p.splits + s];
      s_inv[h] = l > 0.f ? p.out_scale / l : 0.f;
    }
    __syncthreads();
    for (int ks = warp; ks < p.steps; ks += kTkWarps) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int r = g + (x & 1) * 8, c = ks * 16 + 2 * t + (x >> 1) * 8;
        const float* m = p.talk + static_cast<int64_t>(h0 + r) * H + c;
        split2(r < rows && c < H ? m[0] * s_inv[c] : 0.f, r < rows && c + 1 < H ? m[1] * s_inv[c + 1] : 0.f, hi[x], lo[x]);
      }
      s_mix[(ks * 2) * 32 + lane] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      s_mix[(ks * 2 + 1) * 32 + lane] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    __syncthreads();
  }
  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  for (int i = 0; i < mine; ++i) {
    cp_async_wait<kTkStages - 2>();
    __syncwarp();
    const unsigned char* stage = stages + (warp * kTkStages + i % kTkStages) * stage_bytes;
    const float* sw = reinterpret_cast<const float*>(stage);
    const uint32_t vd = ring + i % kTkStages * stage_bytes + w_bytes;
    float w[2][4] = {};
#pragma unroll 1
    for (int ks = 0; ks < p.steps; ++ks) {
      const uint4 h4 = s_mix[(ks * 2) * 32 + lane], l4 = s_mix[(ks * 2 + 1) * 32 + lane];
      const uint32_t hi[4] = {h4.x, h4.y, h4.z, h4.w}, lo[4] = {l4.x, l4.y, l4.z, l4.w};
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const float* e = sw + (ks * 16 + 2 * t + x * 8) * kTkRow + n * 8 + g;
          split2(e[0], e[kTkRow], bh[x], bl[x]);
        }
        Mma::run(w[n], hi, bh[0], bh[1]);
        Mma::run(w[n], lo, bh[0], bh[1]);
        Mma::run(w[n], hi, bl[0], bl[1]);
      }
    }
    uint32_t pa[4], pl[4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) split2(w[n][2 * half], w[n][2 * half + 1], pa[2 * n + half], pl[2 * n + half]);
    const int r = (lane & 7) + (((lane >> 3) & 1) << 3), csel = lane >> 4;
#pragma unroll
    for (int jp = 0; jp < NT / 2; ++jp) {
      uint32_t vb[4];
      ldmatrix_x4_trans(vb, vd + r * (VD * 2) + (((2 * jp + csel) ^ (r & 7)) << 4));
      Mma::run(o[2 * jp], pa, vb[0], vb[1]);
      Mma::run(o[2 * jp + 1], pa, vb[2], vb[3]);
      Mma::run(o[2 * jp], pl, vb[0], vb[1]);
      Mma::run(o[2 * jp + 1], pl, vb[2], vb[3]);
    }
    __syncwarp();
    issue(i + kTkStages - 1);
  }
  cp_async_wait<0>();
  __syncthreads();                       // the rings are idle
  float* sO = reinterpret_cast<float*>(stages);
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    *reinterpret_cast<float2*>(sO + (warp * 16 + g) * kStride + j * 8 + 2 * t) = make_float2(o[j][0], o[j][1]);
    *reinterpret_cast<float2*>(sO + (warp * 16 + g + 8) * kStride + j * 8 + 2 * t) = make_float2(o[j][2], o[j][3]);
  }
  __syncthreads();
  const int half = p.vdim / 2;
  for (int i = tid; i < rows * half; i += kTkThreads) {
    const int r = i / half, d = (i - r * half) * 2, h = h0 + r;
    float2 acc = make_float2(0.f, 0.f);
#pragma unroll
    for (int w = 0; w < kTkWarps; ++w) {
      const float2 x = *reinterpret_cast<const float2*>(sO + (w * 16 + r) * kStride + d);
      acc.x += x.x;
      acc.y += x.y;
    }
    if (p.splits == 1)
      *reinterpret_cast<__nv_bfloat162*>(p.out + b * p.out_stride + static_cast<int64_t>(h) * p.vdim + d) = __floats2bfloat162_rn(acc.x, acc.y);
    else
      *reinterpret_cast<float2*>(p.part + ((static_cast<int64_t>(b) * p.splits + split) * H + h) * p.vdim + d) = acc;
  }
}

__global__ void __launch_bounds__(128) talk_join_kernel(const TalkParams p) {
  const int n = p.heads * p.vdim, i = (blockIdx.x * 128 + threadIdx.x) * 2, b = blockIdx.y;
  if (i >= n) return;
  const float* src = p.part + static_cast<int64_t>(b) * p.splits * n + i;
  float2 acc = make_float2(0.f, 0.f);
  for (int s = 0; s < p.splits; ++s) {
    const float2 x = *reinterpret_cast<const float2*>(src + static_cast<int64_t>(s) * n);
    acc.x += x.x;
    acc.y += x.y;
  }
  *reinterpret_cast<__nv_bfloat162*>(p.out + b * p.out_stride + i) = __floats2bfloat162_rn(acc.x, acc.y);
}

// Pieces per sequence: enough CTAs to fill the GPU twice, none of less than 64 keys.  Depends on shapes only.
static int talk_splits(int batch, int heads, int kv_heads, int64_t most_keys) {
  const int64_t units = static_cast<int64_t>(batch) * kv_heads * ((heads / kv_heads + 15) / 16);
  const int64_t want = (3 * kNumSMs + units - 1) / std::max<int64_t>(units, 1);
  return static_cast<int>(std::max<int64_t>(1, std::min<int64_t>({want, most_keys / 64, 64})));
}
struct TalkScratch {
  int64_t keys, weights, sums, part;
  TalkScratch(int batch, int heads, int vdim, int splits, int64_t most_keys) {
    keys = (most_keys + 15) / 16 * 16;
    weights = static_cast<int64_t>(batch) * heads * keys;
    sums = (static_cast<int64_t>(batch) * heads * splits + 3) / 4 * 4;
    part = splits > 1 ? static_cast<int64_t>(batch) * splits * heads * vdim : 0;
  }
  int64_t bytes() const { return (weights + sums + part) * 4; }
};

// ------------------------------------------------------------------------------------------------ mixture of results
constexpr int kHmThreads = 256;
// a: (tokens, heads, kv_heads, vdim); a thread makes R heads' results of a value head, V columns each.
template <typename TI, typename T, int V, int R>
__global__ void __launch_bounds__(kHmThreads) head_mix_kernel(T* __restrict__ out, int64_t out_stride, const TI* __restrict__ a, const float* __restrict__ talk,
                                                              float out_scale, int64_t tokens, int heads, int kv_heads, int vdim) {
  extern __shared__ float s_talk[];
  for (int i = threadIdx.x; i < heads * heads; i += kHmThreads) s_talk[i] = talk[i] * out_scale;
  __syncthreads();
  const int group = heads / kv_heads, parts = (group + R - 1) / R, cols = vdim / V, per = kv_heads * parts * cols;
  const int64_t items = tokens * per;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * kHmThreads + threadIdx.x; i < items; i += static_cast<int64_t>(gridDim.x) * kHmThreads) {
    const int64_t t = i / per;
    const int x = static_cast<int>(i - t * per), d = x % cols * V, part = x / cols % parts, c = x / (cols * parts);
    const int h0 = c * group + part * R, n = min(R, group - part * R);
    const TI* src = a + (t * heads * kv_heads + c) * vdim + d;
    float acc[R][V];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int e = 0; e < V; ++e) acc[r][e] = 0.f;
#pragma unroll 4
    for (int g = 0; g < heads; ++g) {
      float v[V];
      Vec<TI, V>::load(src + static_cast<int64_t>(g) * kv_heads * vdim, v);
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const float w = s_talk[(h0 + min(r, n - 1)) * heads + g];
#pragma unroll
        for (int e = 0; e < V; ++e) acc[r][e] = fmaf(w, v[e], acc[r][e]);
      }
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (r < n) Vec<T, V>::store(out + t * out_stride + static_cast<int64_t>(h0 + r) * vdim + d, acc[r]);
  }
}

}  // namespace mv

static int check_talk(const char* what, int heads, int kv_heads, int dim, int vdim, float cap) {
  using namespace mv;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || !(cap > 0.f))
    return fail(MV_ERR_SHAPE, "%s: heads %d over %d, dim %d, vdim %d, cap %f", what, heads, kv_heads, dim, vdim, cap);
  return MV_OK;
}

// Bytes of scratch, or -1 when the kernels do not take the sizes or the cap.
extern "C" int64_t mv_talk_decode_workspace_bytes(int batch, int heads, int kv_heads, int dim, int vdim, float cap, int64_t most_keys) {
  using namespace mv;
  if (batch < 0 || batch > 65535 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || heads > 256 || dim <= 0 || vdim <= 0 || dim % 8 ||
      vdim % 8 || dim > 256 || vdim > 256 || !(cap > 0.f && cap <= kTalkCap) || most_keys <= 0)
    return -1;
  const int vd = vdim <= 64 ? 64 : vdim <= 128 ? 128 : 256;
  if (talk_values_smem(vd, (heads + 15) / 16) > 227 * 1024) return -1;
  return TalkScratch(batch, heads, vdim, talk_splits(batch, heads, kv_heads, most_keys), most_keys).bytes();
}

extern "C" int mv_talk_decode(void* out, int64_t out_stride, const void* q, int64_t q_stride, const void* cache,
                              const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size,
                              int64_t num_blocks, const int64_t* positions, const float* r1, const float* r2,
                              const float* talk, float cap, int batch, int heads, int kv_heads, int dim, int vdim,
                              float scale, float out_scale, void* workspace, int64_t workspace_bytes, void* stream) {
  using namespace mv;
  const int rc = check_talk("talk_decode", heads, kv_heads, dim, vdim, cap);
  if (rc) return rc;
  if (max_blocks <= 0 || block_size <= 0) return fail(MV_ERR_SHAPE, "talk_decode: %d blocks of %d", max_blocks, block_size);
  const int64_t most = static_cast<int64_t>(max_blocks) * block_size;
  const int64_t need = mv_talk_decode_workspace_bytes(batch, heads, kv_heads, dim, vdim, cap, most);
  if (need < 0) return fail(MV_ERR_LIMIT, "talk_decode: heads %d, dim %d, vdim %d, cap %f, batch %d", heads, dim, vdim, cap, batch);
  if (batch == 0) return MV_OK;
  if (!out || !q || !cache || !block_tables || !positions || !r1 || !r2 || !talk) return fail(MV_ERR_NULL, "talk_decode: null pointer");
  if (!aligned16(cache) || (reinterpret_cast<uintptr_t>(q) & 3u) || (reinterpret_cast<uintptr_t>(out) & 3u) || q_stride % 2 || out_stride % 2)
    return fail(MV_ERR_ALIGN, "talk_decode: alignment");
  if (!workspace || !aligned16(workspace) || workspace_bytes < need) return fail(MV_ERR_WORKSPACE, "talk_decode: workspace");
  TalkParams p{};
  p.out = static_cast<__nv_bfloat16*>(out); p.out_stride = out_stride; p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_stride;
  p.cache = static_cast<const __nv_bfloat16*>(cache);
  p.tables = block_tables; p.bt_stride = bt_stride; p.max_blocks = max_blocks; p.block_size = block_size; p.num_blocks = num_blocks;
  p.positions = positions; p.r1 = r1; p.r2 = r2; p.talk = talk; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim;
  p.scale = scale; p.cap = cap; p.out_scale = out_scale;
  p.splits = talk_splits(batch, heads, kv_heads, most);
  p.steps = (heads + 15) / 16;
  const TalkScratch sc(batch, heads, vdim, p.splits, most);
  p.keys = sc.keys;
  p.weights = static_cast<float*>(workspace);
  p.sums = p.weights + sc.weights;
  p.part = p.sums + sc.sums;
  auto st = static_cast<cudaStream_t>(stream);
  const dim3 grid(p.splits, kv_heads * ((heads / kv_heads + 15) / 16), batch);
  auto launch = [&](auto kernel, int smem) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "talk_decode: %s", cudaGetErrorString(e));
    kernel<<<grid, kTkThreads, smem, st>>>(p);
    return check_launch("talk_decode");
  };
  auto scores = [&](auto kd) { return launch(talk_scores_kernel<decltype(kd)::value>, kTkWarps * kTkStages * kTkTile * decltype(kd)::value * 2); };
  auto values = [&](auto vd) { return launch(talk_values_kernel<decltype(vd)::value>, talk_values_smem(decltype(vd)::value, p.steps)); };
  using std::integral_constant;
  int r = dim <= 64 ? scores(integral_constant<int, 64>{}) : dim <= 128 ? scores(integral_constant<int, 128>{}) : scores(integral_constant<int, 256>{});
  if (r) return r;
  r = vdim <= 64 ? values(integral_constant<int, 64>{}) : vdim <= 128 ? values(integral_constant<int, 128>{}) : values(integral_constant<int, 256>{});
  if (r || p.splits == 1) return r;
  talk_join_kernel<<<dim3((heads * vdim / 2 + 127) / 128, batch), 128, 0, st>>>(p);
  return check_launch("talk_join");
}

extern "C" int mv_head_mix(void* out, int64_t out_stride, const void* a, int a_dtype, const float* talk, float out_scale,
                           int64_t tokens, int heads, int kv_heads, int vdim, int dtype, void* stream) {
  using namespace mv;
  if ((dtype != MV_BF16 && dtype != MV_F32) || (a_dtype != MV_F32 && a_dtype != dtype)) return fail(MV_ERR_DTYPE, "head_mix: dtypes %d, %d", a_dtype, dtype);
  const int rc = check_talk("head_mix", heads, kv_heads, 1, vdim, 1.f);
  if (rc) return rc;
  if (heads > 240) return fail(MV_ERR_LIMIT, "head_mix: %d heads (at most 240)", heads);
  if (tokens <= 0) return tokens < 0 ? fail(MV_ERR_SHAPE, "head_mix: tokens") : static_cast<int>(MV_OK);
  if (!out || !a || !talk) return fail(MV_ERR_NULL, "head_mix: null pointer");
  auto run = [&](auto in, auto tag) {
    using TI = decltype(in);
    using T = decltype(tag);
    auto go = [&](auto vv, auto rr) {
      constexpr int V = decltype(vv)::value, R = decltype(rr)::value;
      const int group = heads / kv_heads;
      const int64_t items = tokens * kv_heads * ((group + R - 1) / R) * (vdim / V);
      const unsigned grid = static_cast<unsigned>(std::min<int64_t>((items + kHmThreads - 1) / kHmThreads, kNumSMs * 16));
      const cudaError_t e = cudaFuncSetAttribute(head_mix_kernel<TI, T, V, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, heads * heads * 4);
      if (e != cudaSuccess) return fail(MV_ERR_CUDA, "head_mix: %s", cudaGetErrorString(e));
      head_mix_kernel<TI, T, V, R><<<grid, kHmThreads, heads * heads * 4, static_cast<cudaStream_t>(stream)>>>(
          static_cast<T*>(out), out_stride, static_cast<const TI*>(a), talk, out_scale, tokens, heads, kv_heads, vdim);
      return check_launch("head_mix");
    };
    using std::integral_constant;
    const int group = heads / kv_heads;
    if (vdim % 8 == 0 && aligned16(a) && vec8_ok(out, out_stride, sizeof(T))) {
      if (group == 1) return go(integral_constant<int, 8>{}, integral_constant<int, 1>{});
      if (group == 2) return go(integral_constant<int, 8>{}, integral_constant<int, 2>{});
      return go(integral_constant<int, 8>{}, integral_constant<int, 4>{});
    }
    return go(integral_constant<int, 1>{}, integral_constant<int, 4>{});
  };
  if (dtype == MV_F32) return run(float{}, float{});
  return a_dtype == MV_F32 ? run(float{}, __nv_bfloat16{}) : run(__nv_bfloat16{}, __nv_bfloat16{});
}
