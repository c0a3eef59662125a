// Decode attention over the paged latent cache, absorbed form, bf16: one query row per sequence and head, all heads
// of a sequence share the cached rows [c | rotated key part], and the value is the c part of the same row, so a row
// that is in shared memory serves the score and the sum.
//
// The batch's 64-key tiles form one stream that is cut into equal ranges, one per persistent CTA (the grid depends on
// shapes only; the cut on the device-side lengths).  A CTA's range may end or begin inside a sequence: those pieces go
// to the workspace as (m, l, unnormalised sum) and latent_combine_kernel joins them; whole sequences are written
// directly.  16 heads per CTA are the 16 rows of m16n8k16 MMAs (the kernel is HBM-bound, and mma.sync needs no wider
// tile); the scores and the softmax are fp32, and the weights enter the product as two bf16 terms (value and rounding
// residue).  The learned sink joins the denominator when a sequence is finished.
//
// HBM-bound: bytes = sum(ctx) * (rank + rot_dim) * 2.
#include <algorithm>
#include "mma.cuh"
#include "vec.cuh"

namespace mv {

constexpr int kLdThreads = 256, kLdWarps = 8;
constexpr int kLdKeys = 64, kLdHeads = 16;
constexpr int kLdMaxSeqs = 1024, kLdMaxRank = 512;
constexpr int kLdSStride = kLdKeys + 4;    // floats per score row
constexpr int kLdPStride = kLdKeys + 8;    // bf16 per weight row

struct LdParams {
  __nv_bfloat16* out; int64_t out_stride, out_head_stride;
  const __nv_bfloat16* q_lat; int64_t q_lat_stride, q_lat_head_stride;
  const __nv_bfloat16* q_rot; int64_t q_rot_stride, q_rot_head_stride;
  const __nv_bfloat16* cache;
  const int32_t* tables; int64_t bt_stride; int max_blocks, block_size; int64_t num_blocks;
  const int64_t* positions;      // keys of sequence b: positions[b] + 1
  const int32_t* active;         // null, or per sequence < 0: a padding row without keys
  const __nv_bfloat16* sink;
  int batch, heads, rank, rot_dim;
  float scale_log2;
  float* ws;                     // [head tile][cta][2] pieces of {m[16], l[16], acc[16][rank]}
};

__host__ __device__ inline int64_t ld_piece_floats(int rank) { return 2 * kLdHeads + static_cast<int64_t>(kLdHeads) * rank; }
__device__ __forceinline__ int ld_tiles(const LdParams& p, int b) {
  if (p.active && p.active[b] < 0) return 0;
  const int64_t n = min(p.positions[b] + 1, static_cast<int64_t>(p.max_blocks) * p.block_size);
  return static_cast<int>((n + kLdKeys - 1) / kLdKeys);
}
// s_start[b] = tiles before sequence b, s_start[batch] = all
__device__ __forceinline__ void ld_prefix(const LdParams& p, int* s_start) {
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
      carry += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (lane == 0) s_start[p.batch] = carry;
  }
  __syncthreads();
}
__device__ __forceinline__ int ld_cut(int total, int c, int ctas) { return static_cast<int>(static_cast<int64_t>(total) * c / ctas); }

__global__ void __launch_bounds__(kLdThreads, 1) latent_decode_kernel(const LdParams p) {
  extern __shared__ __align__(128) unsigned char raw[];
  __shared__ int s_start[kLdMaxSeqs + 1];
  __shared__ float s_m[kLdHeads], s_l[kLdHeads], s_c[kLdHeads];
  const int R = p.rank + p.rot_dim, row_bytes = R * 2 + 16;
  unsigned char* kv = raw;                                   // [2][64][row_bytes]
  unsigned char* sq = kv + 2 * kLdKeys * row_bytes;          // [16][row_bytes]
  float* ss = reinterpret_cast<float*>(sq + kLdHeads * row_bytes);                       // [16][kLdSStride]
  __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(ss + kLdHeads * kLdSStride);      // [2][16][kLdPStride]
  const uint32_t kv_s = smem_u32(kv), q_s = smem_u32(sq), p_s = smem_u32(sp);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h0 = blockIdx.y * kLdHeads, nh = min(kLdHeads, p.heads - h0);
  ld_prefix(p, s_start);
  const int total = s_start[p.batch], ctas = gridDim.x, c = blockIdx.x;
  const int g0 = ld_cut(total, c, ctas), g1 = ld_cut(total, c + 1, ctas);
  if (g0 >= g1) return;

  auto find = [&](int g) {      // the sequence of tile g: last b with s_start[b] <= g and a tile of its own
    int lo = 0, hi = p.batch - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (s_start[mid] <= g) lo = mid; else hi = mid - 1;
    }
    return lo;
  };
  const int chunks = R / 8;
  int load_b = find(g0);
  auto load = [&](int g, int buf) {
    if (g < g1) {
      while (g >= s_start[load_b + 1]) ++load_b;
      const int k0 = (g - s_start[load_b]) * kLdKeys;
      const int64_t n = min(p.positions[load_b] + 1, static_cast<int64_t>(p.max_blocks) * p.block_size);
      const int32_t* table = p.tables + static_cast<int64_t>(load_b) * p.bt_stride;
#pragma unroll
      for (int i = 0; i < kLdKeys / kLdWarps; ++i) {
        const int r = i * kLdWarps + warp, pos = k0 + r, blk = pos / p.block_size;
        const int32_t phys = pos < n ? table[blk] : -1;
        const bool ok = phys >= 0 && phys < p.num_blocks;
        const __nv_bfloat16* src = p.cache + (static_cast<int64_t>(ok ? phys : 0) * p.block_size + (ok ? pos - blk * p.block_size : 0)) * R;
        const uint32_t dst = kv_s + (buf * kLdKeys + r) * row_bytes;
        for (int ch = lane; ch < chunks; ch += 32) cp_async16(dst + ch * 16, src + ch * 8, ok ? 16 : 0);
      }
    }
    cp_async_commit();
  };
  load(g0, 0);
  load(g0 + 1, 1);

  const int nv = p.rank / 64;          // 8-column tiles of the sum per warp
  const int vbase = warp * nv * 8;
  float acc[kLdMaxRank / 64][4];
  int b = find(g0), first_g = g0;
  bool fresh = true;
  int64_t nkeys = 0;
  for (int g = g0; g < g1; ++g) {
    const int buf = (g - g0) & 1;
    while (g >= s_start[b + 1]) ++b;
    if (fresh) {
      first_g = g;
      nkeys = min(p.positions[b] + 1, static_cast<int64_t>(p.max_blocks) * p.block_size);
      for (int i = tid; i < kLdHeads * chunks; i += kLdThreads) {
        const int h = i / chunks, col = (i - h * chunks) * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (h < nh)
          v = *reinterpret_cast<const uint4*>(col < p.rank ? p.q_lat + b * p.q_lat_stride + (h0 + h) * p.q_lat_head_stride + col
                                                           : p.q_rot + b * p.q_rot_stride + (h0 + h) * p.q_rot_head_stride + col - p.rank);
        *reinterpret_cast<uint4*>(sq + h * row_bytes + col * 2) = v;
      }
      if (tid < kLdHeads) { s_m[tid] = -INFINITY; s_l[tid] = 0.f; }
#pragma unroll
      for (int i = 0; i < kLdMaxRank / 64; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
      fresh = false;
    }
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t kb = kv_s + buf * kLdKeys * row_bytes;
    {  // scores of 8 keys per warp
      float d[4][4] = {};
      const uint32_t qa = q_s + ((lane & 7) + ((lane >> 3) & 1) * 8) * row_bytes + (lane >> 4) * 16;
      const uint32_t ka = kb + (warp * 8 + (lane & 7)) * row_bytes + (lane >> 3) * 16;
#pragma unroll 2
      for (int k = 0; k < R; k += 64) {
        uint32_t a[4], kf[4];
        ldmatrix_x4(kf, ka + k * 2);
        ldmatrix_x4(a, qa + k * 2);
        Mma16816<__nv_bfloat16>::run(d[0], a, kf[0], kf[1]);
        ldmatrix_x4(a, qa + k * 2 + 32);
        Mma16816<__nv_bfloat16>::run(d[1], a, kf[2], kf[3]);
        if (k + 32 < R) {
          ldmatrix_x4(kf, ka + k * 2 + 64);
          ldmatrix_x4(a, qa + k * 2 + 64);
          Mma16816<__nv_bfloat16>::run(d[2], a, kf[0], kf[1]);
          ldmatrix_x4(a, qa + k * 2 + 96);
          Mma16816<__nv_bfloat16>::run(d[3], a, kf[2], kf[3]);
        }
      }
      const int r = lane >> 2, col = warp * 8 + (lane & 3) * 2;
      const int64_t key = static_cast<int64_t>(g - s_start[b]) * kLdKeys + col;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float v = (d[0][j] + d[1][j]) + (d[2][j] + d[3][j]);
        const int cc = col + (j & 1);
        ss[(r + (j >> 1) * 8) * kLdSStride + cc] = key + (j & 1) < nkeys ? v * p.scale_log2 : -INFINITY;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {        // two rows per warp
      const int h = warp * 2 + i;
      const float a = ss[h * kLdSStride + lane], e = ss[h * kLdSStride + lane + 32];
      float mx = fmaxf(a, e);
#pragma unroll
      for (int o = 16; o; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_old = s_m[h], m_new = fmaxf(m_old, mx);
      const float pa = m_new == -INFINITY ? 0.f : exp2f(a - m_new), pe = m_new == -INFINITY ? 0.f : exp2f(e - m_new);
      const float sum = warp_sum(pa + pe);
      const __nv_bfloat16 ha = __float2bfloat16_rn(pa), he = __float2bfloat16_rn(pe);
      sp[h * kLdPStride + lane] = ha;
      sp[h * kLdPStride + lane + 32] = he;
      sp[(kLdHeads + h) * kLdPStride + lane] = __float2bfloat16_rn(pa - __bfloat162float(ha));
      sp[(kLdHeads + h) * kLdPStride + lane + 32] = __float2bfloat16_rn(pe - __bfloat162float(he));
      if (lane == 0) {
        const float corr = m_new == -INFINITY ? 1.f : exp2f(m_old - m_new);
        s_c[h] = corr;
        s_l[h] = s_l[h] * corr + sum;
        s_m[h] = m_new;
      }
    }
    __syncthreads();
    {  // weighted sum: this warp's columns of all 64 keys
      const float c0 = s_c[lane >> 2], c1 = s_c[(lane >> 2) + 8];
#pragma unroll
      for (int i = 0; i < kLdMaxRank / 64; ++i) {
        acc[i][0] *= c0; acc[i][1] *= c0; acc[i][2] *= c1; acc[i][3] *= c1;
      }
      const uint32_t pa = p_s + (((lane & 7) + ((lane >> 3) & 1) * 8) * kLdPStride + (lane >> 4) * 8) * 2;
      const uint32_t va = kb + ((lane & 7) + ((lane >> 3) & 1) * 8) * row_bytes + (vbase + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int k = 0; k < kLdKeys; k += 16) {
        uint32_t hi[4], lo[4];
        ldmatrix_x4(hi, pa + k * 2);
        ldmatrix_x4(lo, pa + kLdHeads * kLdPStride * 2 + k * 2);
#pragma unroll
        for (int i = 0; i < kLdMaxRank / 64; i += 2) {
          if (i < nv) {
            uint32_t v[4];
            ldmatrix_x4_trans(v, va + k * row_bytes + i * 16);
            Mma16816<__nv_bfloat16>::run(acc[i], hi, v[0], v[1]);
            Mma16816<__nv_bfloat16>::run(acc[i], lo, v[0], v[1]);
            if (i + 1 < nv) {
              Mma16816<__nv_bfloat16>::run(acc[i + 1], hi, v[2], v[3]);
              Mma16816<__nv_bfloat16>::run(acc[i + 1], lo, v[2], v[3]);
            }
          }
        }
      }
    }
    __syncthreads();           // the buffer, the weights and the row statistics are free again
    load(g + 2, buf);
    const bool last = g + 1 == s_start[b + 1];
    if (last || g + 1 == g1) {
      const bool whole = last && first_g == s_start[b];
      const int r = lane >> 2, col = (lane & 3) * 2;
      if (whole) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int h = r + half * 8;
          if (h >= nh) continue;
          float m = s_m[h], l = s_l[h], f = 1.f;
          if (p.sink) {
            const float sk = __bfloat162float(p.sink[h0 + h]) * 1.4426950408889634f, mm = fmaxf(m, sk);
            f = exp2f(m - mm);
            l = l * f + exp2f(sk - mm);
          }
          const float inv = l > 0.f ? f / l : 0.f;
          __nv_bfloat16* o = p.out + b * p.out_stride + (h0 + h) * p.out_head_stride + vbase + col;
#pragma unroll
          for (int i = 0; i < kLdMaxRank / 64; ++i)
            if (i < nv)
              *reinterpret_cast<__nv_bfloat162*>(o + i * 8) = __floats2bfloat162_rn(acc[i][half * 2] * inv, acc[i][half * 2 + 1] * inv);
        }
      } else {
        float* piece = p.ws + ((static_cast<int64_t>(blockIdx.y) * ctas + c) * 2 + (first_g == g0 ? 0 : 1)) * ld_piece_floats(p.rank);
        if (tid < kLdHeads) { piece[tid] = s_m[tid]; piece[kLdHeads + tid] = s_l[tid]; }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          float* o = piece + 2 * kLdHeads + (r + half * 8) * p.rank + vbase + col;
#pragma unroll
          for (int i = 0; i < kLdMaxRank / 64; ++i)
            if (i < nv) *reinterpret_cast<float2*>(o + i * 8) = make_float2(acc[i][half * 2], acc[i][half * 2 + 1]);
        }
      }
      __syncthreads();         // s_m / s_l are read before the next sequence resets them
      fresh = true;
    }
  }
}

// One CTA per (sequence, head): joins the pieces of a sequence that several CTAs worked on.  Sequences without keys
// (padding rows) get zeros.
__global__ void __launch_bounds__(128) latent_combine_kernel(const LdParams p, int ctas) {
  __shared__ int s_start[kLdMaxSeqs + 1];
  ld_prefix(p, s_start);
  const int b = blockIdx.x, h = blockIdx.y, total = s_start[p.batch], t0 = s_start[b], t1 = s_start[b + 1];
  __nv_bfloat16* o = p.out + b * p.out_stride + h * p.out_head_stride;
  if (t0 == t1) {
    for (int d = threadIdx.x; d < p.rank; d += 128) o[d] = __float2bfloat16_rn(0.f);
    return;
  }
  auto cta_of = [&](int g) {
    int c = static_cast<int>(static_cast<int64_t>(g) * ctas / total);
    while (c + 1 < ctas && ld_cut(total, c + 1, ctas) <= g) ++c;
    while (c > 0 && ld_cut(total, c, ctas) > g) --c;
    return c;
  };
  const int c0 = cta_of(t0), c1 = cta_of(t1 - 1);
  if (c0 == c1) return;        // written whole
  const int64_t pf = ld_piece_floats(p.rank);
  const float* base = p.ws + static_cast<int64_t>(h / kLdHeads) * ctas * 2 * pf;
  const int r = h % kLdHeads;
  auto piece = [&](int c) { return base + (c * 2 + (c == c0 && ld_cut(total, c, ctas) != t0 ? 1 : 0)) * pf; };
  // CTAs whose range is empty (fewer tiles than CTAs) have no piece
  const float sk = p.sink ? __bfloat162float(p.sink[h]) * 1.4426950408889634f : -INFINITY;
  float m = sk;
  for (int c = c0; c <= c1; ++c)
    if (ld_cut(total, c, ctas) < ld_cut(total, c + 1, ctas)) m = fmaxf(m, piece(c)[r]);
  float l = p.sink ? exp2f(sk - m) : 0.f;
  for (int c = c0; c <= c1; ++c)
    if (ld_cut(total, c, ctas) < ld_cut(total, c + 1, ctas)) l += piece(c)[kLdHeads + r] * exp2f(piece(c)[r] - m);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int d = threadIdx.x; d < p.rank; d += 128) {
    float a = 0.f;
    for (int c = c0; c <= c1; ++c)
      if (ld_cut(total, c, ctas) < ld_cut(total, c + 1, ctas)) {
        const float* q = piece(c);
        a = fmaf(q[2 * kLdHeads + r * p.rank + d], exp2f(q[r] - m), a);
      }
    o[d] = __float2bfloat16_rn(a * inv);
  }
}

static bool ld_takes(int batch, int rank, int rot_dim) {
  return batch <= kLdMaxSeqs && rank % 64 == 0 && rank <= kLdMaxRank && rot_dim % 32 == 0 && rank + rot_dim <= 640;
}
static int ld_ctas(int heads) { return std::max(1, kNumSMs / ((heads + kLdHeads - 1) / kLdHeads)); }

}  // namespace mv

extern "C" int64_t mv_latent_decode_workspace_bytes(int batch, int heads, int rank, int rot_dim) {
  using namespace mv;
  if (batch < 0 || heads <= 0 || rank <= 0 || rot_dim < 0 || !ld_takes(batch, rank, rot_dim)) return -1;
  return static_cast<int64_t>((heads + kLdHeads - 1) / kLdHeads) * ld_ctas(heads) * 2 * ld_piece_floats(rank) * 4;
}

extern "C" int mv_latent_decode(void* out, int64_t out_stride, int64_t out_head_stride, const void* q_lat,
                                int64_t q_lat_stride, int64_t q_lat_head_stride, const void* q_rot,
                                int64_t q_rot_stride, int64_t q_rot_head_stride, const void* cache,
                                const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size,
                                int64_t num_blocks, const int64_t* positions, const int32_t* active, const void* sink,
                                int batch, int heads, int rank, int rot_dim, float scale, void* workspace,
                                int64_t workspace_bytes, void* stream) {
  using namespace mv;
  if (batch < 0 || heads <= 0 || block_size <= 0 || max_blocks < 0) return fail(MV_ERR_SHAPE, "latent_decode: batch %d heads %d", batch, heads);
  if (!ld_takes(batch, rank, rot_dim)) return fail(MV_ERR_LIMIT, "latent_decode: batch %d rank %d rot_dim %d", batch, rank, rot_dim);
  if (batch == 0) return MV_OK;
  if (!out || !q_lat || (rot_dim && !q_rot) || !cache || !block_tables || !positions || !workspace)
    return fail(MV_ERR_NULL, "latent_decode: null pointer");
  if (workspace_bytes < mv_latent_decode_workspace_bytes(batch, heads, rank, rot_dim)) return fail(MV_ERR_WORKSPACE, "latent_decode: workspace");
  if (!vec8_ok(q_lat, q_lat_stride, 2) || q_lat_head_stride % 8 || !vec8_ok(q_rot, q_rot_stride, 2) || q_rot_head_stride % 8 ||
      !aligned16(cache) || !vec8_ok(out, out_stride, 2) || out_head_stride % 8 || !aligned16(workspace))
    return fail(MV_ERR_ALIGN, "latent_decode: rows must start on 16-byte boundaries");
  LdParams p{static_cast<__nv_bfloat16*>(out), out_stride, out_head_stride, static_cast<const __nv_bfloat16*>(q_lat),
             q_lat_stride, q_lat_head_stride, static_cast<const __nv_bfloat16*>(q_rot), q_rot_stride, q_rot_head_stride,
             static_cast<const __nv_bfloat16*>(cache), block_tables, bt_stride, max_blocks, block_size, num_blocks,
             positions, active, static_cast<const __nv_bfloat16*>(sink), batch, heads, rank, rot_dim,
             scale * 1.4426950408889634f, static_cast<float*>(workspace)};
  const int row_bytes = (rank + rot_dim) * 2 + 16;
  const size_t smem = static_cast<size_t>(2 * kLdKeys + kLdHeads) * row_bytes + kLdHeads * kLdSStride * 4 + 2 * kLdHeads * kLdPStride * 2;
  const cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return fail(MV_ERR_CUDA, "latent_decode: %s", cudaGetErrorString(e));
  const int ctas = ld_ctas(heads);
  auto st = static_cast<cudaStream_t>(stream);
  latent_decode_kernel<<<dim3(ctas, (heads + kLdHeads - 1) / kLdHeads), kLdThreads, smem, st>>>(p);
  latent_combine_kernel<<<dim3(batch, heads), 128, 0, st>>>(p, ctas);
  return check_launch("latent_decode");
}
