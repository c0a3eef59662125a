// Gated linear attention and time mixing in chunks of 64 tokens.  With b_t the running sums of the channels' log2 decays inside the chunk:
//   O = (q 2^b) S_0 + A V,      A[t, j] = sum_k q_t k_j 2^(b_t - b_j), j <= t
//   S = 2^b_last S_0 + (k 2^(b_last - b))^T V
// Time mixing (kTime) reads the state before the token's own decay: b_(t-1) in the place of b_t beside q, j < t in A, whose
// diagonal is q_t . (u k_t).
// gla_prepare_kernel  per chunk and head: b, both decayed operands, A.  A's 16 x 16 blocks are products of factors taken
//                     against b at one token, on tensor cores in two terms each.  Below the diagonal that is the last token
//                     before the block's rows, and every power of two is at most one.  On the diagonal it is the block's
//                     middle; a block in which some channel forgets more than 2^-60 is summed channel by channel instead.
// gla_chunk_kernel    per sequence, head and block of value columns: see state_chunk.cuh
// V enters as the projection left it; the decayed operands, A and S in two terms.
#include "state_chunk.cuh"

namespace mv {

constexpr int kGpThreads = 256;

struct GlaChunkParams {
  __nv_bfloat16* out; int64_t out_stride;
  const __nv_bfloat16 *q, *k, *v; int64_t stride;
  const __nv_bfloat16* z; int64_t z_stride;
  float inv_tau, q_scale;
  const float* zf; const __nv_bfloat16 *w0, *bonus;      // time mixing: z in fp32, its offset and the bonus (heads, K)
  const int32_t *cu, *slots, *start;
  int num_seqs;
  float* state; int num_slots, heads, K, V;
  unsigned char* scratch;                       // [chunk][head][Q hi, Q lo, K hi, K lo, A hi, A lo, 2^b_last]
};

template <int K> struct GlaScratch {
  static constexpr int64_t kVec = kChunk * K, kA = 4 * kVec, kDecay = kA + 2 * kChunk * kChunk;     // offsets in elements
  static constexpr int64_t kBytes = kDecay * 2 + K * 4;
};

template <int K> struct GlaPrepShape {
  static constexpr int kRow = K + 8, kB = K + 4;
  static constexpr int kBytes = 2 * kChunk * kRow * 2 + (kChunk + 1) * kB * 4 + kChunk * 4;
};

template <int K, bool kTime>
__global__ void __launch_bounds__(kGpThreads) gla_prepare_kernel(const GlaChunkParams p) {
  using Sh = GlaPrepShape<K>;
  using Sc = GlaScratch<K>;
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16 *sQ = reinterpret_cast<__nv_bfloat16*>(smem), *sK = sQ + kChunk * Sh::kRow;
  float* sB = reinterpret_cast<float*>(sK + kChunk * Sh::kRow) + Sh::kB;     // a row of zeros in front of token 0
  float* sOwn = sB + kChunk * Sh::kB;                                        // A's diagonal, time mixing
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y;
  int seq, chunk;
  if (!find_chunk(p.cu, p.num_seqs, blockIdx.x, seq, chunk)) return;     // uniform: the grid is an upper bound
  const int64_t first = p.cu[seq] + static_cast<int64_t>(chunk) * kChunk;
  const int nt = min(kChunk, static_cast<int>(p.cu[seq + 1] - first));
  __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.scratch + (static_cast<int64_t>(blockIdx.x) * p.heads + h) * Sc::kBytes);
  {
    const uint32_t qd = smem_u32(sQ), kd = smem_u32(sK);
    for (int i = tid; i < kChunk * (K / 8); i += kGpThreads) {
      const int r = i / (K / 8), c = (i % (K / 8)) * 8;
      const bool ok = r < nt && c < p.K;
      const int64_t off = ok ? (first + r) * p.stride + h * p.K + c : 0;
      cp_async16(qd + (r * Sh::kRow + c) * 2, p.q + off, ok ? 16 : 0);
      cp_async16(kd + (r * Sh::kRow + c) * 2, p.k + off, ok ? 16 : 0);
    }
    cp_async_commit();
  }
  for (int i = tid; i < kChunk * K; i += kGpThreads) {
    const int r = i / K, c = i % K;
    const int64_t at = (first + r) * p.z_stride + h * p.K + c;
    float b = 0.f;
    if (r < nt && c < p.K)
      b = kTime ? time_log_decay(p.zf[at] + __bfloat162float(p.w0[h * p.K + c])) : channel_log_decay(__bfloat162float(p.z[at]), p.inv_tau);
    sB[r * Sh::kB + c] = b * kLog2e;
  }
  for (int c = tid; c < Sh::kB; c += kGpThreads) sB[c - Sh::kB] = 0.f;
  __syncthreads();
  for (int i = tid; i < 4 * K; i += kGpThreads) {        // running sums of 16 tokens
    float* b = sB + (i / K) * 16 * Sh::kB + i % K;
    float run = 0.f;
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      run += b[r * Sh::kB];
      b[r * Sh::kB] = run;
    }
  }
  __syncthreads();
  for (int c = tid; c < K; c += kGpThreads) {            // ... joined
    float run = sB[15 * Sh::kB + c];
#pragma unroll
    for (int blk = 1; blk < 4; ++blk) {
      const float mine = sB[(blk * 16 + 15) * Sh::kB + c];
#pragma unroll
      for (int r = 0; r < 16; ++r) sB[(blk * 16 + r) * Sh::kB + c] += run;
      run += mine;
    }
    reinterpret_cast<float*>(dst + Sc::kDecay)[c] = fast_exp2(sB[(kChunk - 1) * Sh::kB + c]);
  }
  cp_async_wait<0>();
  __syncthreads();
  if (kTime) {
    for (int t = warp; t < kChunk; t += kGpThreads / 32) {
      float own = 0.f;
      for (int c = lane; c < p.K; c += 32)
        own = fmaf(__bfloat162float(sQ[t * Sh::kRow + c]) * __bfloat162float(p.bonus[h * p.K + c]), __bfloat162float(sK[t * Sh::kRow + c]), own);
      own = warp_sum(own);
      if (lane == 0) sOwn[t] = own;
    }
    __syncthreads();
  }
  const float* sE = kTime ? sB - Sh::kB : sB;            // exponents beside q
  {
    uint32_t* o = reinterpret_cast<uint32_t*>(dst);
    for (int i = tid; i < kChunk * K / 2; i += kGpThreads) {
      const int r = i / (K / 2), c = (i % (K / 2)) * 2;
      const float2 b = *reinterpret_cast<const float2*>(sB + r * Sh::kB + c), e = *reinterpret_cast<const float2*>(sE + r * Sh::kB + c);
      const float2 last = *reinterpret_cast<const float2*>(sB + (kChunk - 1) * Sh::kB + c);
      const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sQ + r * Sh::kRow + c));
      const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sK + r * Sh::kRow + c));
      uint32_t hi, lo;
      split2(q.x * p.q_scale * fast_exp2(e.x), q.y * p.q_scale * fast_exp2(e.y), hi, lo);
      o[i] = hi;
      o[Sc::kVec / 2 + i] = lo;
      split2(k.x * fast_exp2(last.x - b.x), k.y * fast_exp2(last.y - b.y), hi, lo);
      o[Sc::kVec + i] = hi;
      o[Sc::kVec * 3 / 2 + i] = lo;
    }
  }
  uint32_t* gA = reinterpret_cast<uint32_t*>(dst + Sc::kA);
  auto put = [&](int t, int j, float x, float y) {
    uint32_t hi, lo;
    split2(x, y, hi, lo);
    gA[(t * kChunk + j) / 2] = hi;
    gA[kChunk * kChunk / 2 + (t * kChunk + j) / 2] = lo;
  };
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  // blocks 0 .. 5 below the diagonal, (1,0) (2,0) (2,1) (3,0) (3,1) (3,2), then the four on it
#pragma unroll 1
  for (int blk = warp; blk < 10; blk += kGpThreads / 32) {
    const bool diag = blk >= 6;
    const int bi = diag ? blk - 6 : blk == 0 ? 1 : blk < 3 ? 2 : 3, bj = diag ? bi : blk - bi * (bi - 1) / 2;
    const float* ref = sB + (diag ? bi * 16 + 7 : bi * 16 - 1) * Sh::kB;
    if (diag) {
      float least = 0.f;
      for (int c = lane; c < K; c += 32)
        least = fminf(least, sB[(bi * 16 + 15) * Sh::kB + c] - (bi ? sB[(bi * 16 - 1) * Sh::kB + c] : 0.f));
      if (__any_sync(0xffffffffu, least < -60.f)) {
        for (int i = lane; i < 16 * 8; i += 32) {        // two neighbouring keys of one token
          const int t = bi * 16 + (i >> 3), j = bi * 16 + (i & 7) * 2;
          const int j_end = kTime ? t - 1 : t;
          float x = 0.f, y = 0.f;
          for (int c = 0; j <= j_end && c < K; ++c) {
            const float q = __bfloat162float(sQ[t * Sh::kRow + c]), bt = sE[t * Sh::kB + c];
            x = fmaf(q * __bfloat162float(sK[j * Sh::kRow + c]), fast_exp2(bt - sB[j * Sh::kB + c]), x);
            if (j + 1 <= j_end) y = fmaf(q * __bfloat162float(sK[(j + 1) * Sh::kRow + c]), fast_exp2(bt - sB[(j + 1) * Sh::kB + c]), y);
          }
          if (kTime) {
            if (j == t) x = sOwn[t];
            if (j + 1 == t) y = sOwn[t];
          }
          put(t, j, x * p.q_scale, y * p.q_scale);
        }
        continue;
      }
    }
    float acc[2][4] = {};
#pragma unroll 2
    for (int kb = 0; kb < K; kb += 16) {
      uint32_t ah[4], al[4], bh[4], bl[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        // A: rows g, g + 8 of the block's tokens, channels c2 and c2 + 8;  B: n-tiles of eight keys each
        const int c = kb + c2 + (x >> 1) * 8, t = bi * 16 + g + (x & 1) * 8;
        const float2 r = *reinterpret_cast<const float2*>(ref + c), b = *reinterpret_cast<const float2*>(sE + t * Sh::kB + c);
        const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sQ + t * Sh::kRow + c));
        split2(q.x * fast_exp2(b.x - r.x), q.y * fast_exp2(b.y - r.y), ah[x], al[x]);
        const int cj = kb + c2 + (x & 1) * 8, j = bj * 16 + g + (x >> 1) * 8;
        const float2 rj = *reinterpret_cast<const float2*>(ref + cj), bb = *reinterpret_cast<const float2*>(sB + j * Sh::kB + cj);
        const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sK + j * Sh::kRow + cj));
        split2(k.x * fast_exp2(rj.x - bb.x), k.y * fast_exp2(rj.y - bb.y), bh[x], bl[x]);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        Mma::run(acc[n], ah, bh[2 * n], bh[2 * n + 1]);
        Mma::run(acc[n], al, bh[2 * n], bh[2 * n + 1]);
        Mma::run(acc[n], ah, bl[2 * n], bl[2 * n + 1]);
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = bi * 16 + g + half * 8, j = bj * 16 + n * 8 + c2;
        float x = acc[n][2 * half], y = acc[n][2 * half + 1];
        if (kTime) {
          if (j == t) x = sOwn[t];
          if (j + 1 == t) y = sOwn[t];
        }
        put(t, j, j <= t ? x * p.q_scale : 0.f, j + 1 <= t ? y * p.q_scale : 0.f);
      }
  }
}

template <int K> struct GlaChunkShape {
  static constexpr int kRow = K + 8;
  static constexpr int kVec = kChunk * kRow * 2, kTile = 2 * kChunk * kCkRow * 2;       // bytes
  static constexpr int stage(int pb) { return 4 * kVec + kChunk * (pb + 8) * 2 + kTile + K * 4; }
};

template <int K>
__global__ void __launch_bounds__(kChunkThreads, 1) gla_chunk_kernel(const GlaChunkParams p, int pb) {
  using Sh = GlaChunkShape<K>;
  using Sc = GlaScratch<K>;
  extern __shared__ __align__(16) unsigned char smem[];
  const int s = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * pb, pw = min(pb, p.V - p0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c2 = (lane & 3) * 2;
  const int vrow = pb + 8;
  const int first = p.cu[s], n_tok = p.cu[s + 1] - first;
  if (n_tok <= 0) return;
  const int chunk0 = chunks_before(p.cu, s), chunks = (n_tok + kChunk - 1) / kChunk;
  const int slot = p.slots[s], st0 = p.start[s];
  const bool live = slot >= 0 && slot < p.num_slots && st0 >= 0;
  float* gS = p.state + (static_cast<int64_t>(live ? slot : 0) * p.heads + h) * p.K * p.V;
  const int stage_bytes = Sh::stage(pb);
  const uint32_t base = smem_u32(smem);
  const __nv_bfloat16* v = p.v + static_cast<int64_t>(h) * p.V + p0;

  auto issue = [&](int c) {
    const uint32_t st = base + (c & 1) * stage_bytes;
    const int64_t row0 = static_cast<int64_t>(first) + c * kChunk;
    const int nt = min(kChunk, n_tok - c * kChunk);
    const __nv_bfloat16* src =
        reinterpret_cast<const __nv_bfloat16*>(p.scratch + (static_cast<int64_t>(chunk0 + c) * p.heads + h) * Sc::kBytes);
    for (int i = tid; i < 4 * kChunk * (K / 8); i += kChunkThreads) {
      const int r = i / (K / 8), cc = (i % (K / 8)) * 8;
      cp_async16(st + (r * Sh::kRow + cc) * 2, src + r * K + cc, 16);
    }
    const uint32_t vd = st + 4 * Sh::kVec, ad = vd + kChunk * vrow * 2;
    for (int i = tid; i < kChunk * (pb / 8); i += kChunkThreads) {
      const int r = i / (pb / 8), cc = (i % (pb / 8)) * 8;
      const bool ok = r < nt && cc < pw;
      cp_async16(vd + (r * vrow + cc) * 2, ok ? v + (row0 + r) * p.stride + cc : p.v, ok ? 16 : 0);
    }
    load_lower(ad, src + Sc::kA, tid, kChunkThreads);
    for (int i = tid; i < K / 4; i += kChunkThreads) cp_async16(ad + Sh::kTile + i * 16, src + Sc::kDecay + i * 8, 16);
    cp_async_commit();
  };
  issue(0);
  const bool work = warp * 16 < pw;
  ChunkState<K> S;
  S.load(gS, p0 + warp * 16, p0 + pw, p.V, p.K, lane, work && live && st0 > 0);
  const LaneAt at(lane);
  for (int c = 0; c < chunks; ++c) {
    cp_async_wait<0>();
    __syncthreads();                     // chunk c is here, and nobody reads the other stage any more
    if (c + 1 < chunks) issue(c + 1);
    if (!work) continue;
    unsigned char* stage = smem + (c & 1) * stage_bytes;
    const uint32_t st = base + (c & 1) * stage_bytes;
    const uint32_t vd = st + 4 * Sh::kVec, ad = vd + kChunk * vrow * 2;
    const float* decay = reinterpret_cast<const float*>(stage + 4 * Sh::kVec + kChunk * vrow * 2 + Sh::kTile);
    uint32_t va[4][4];                   // V^T, the A operand of two products
#pragma unroll
    for (int ib = 0; ib < 4; ++ib) ldmatrix_x4_trans(va[ib], vd + ((ib * 16 + at.row_b) * vrow + warp * 16 + at.col_b) * 2);
    float O[8][4] = {};
#pragma unroll
    for (int kb = 0; kb < K / 16; ++kb) {        // S_0^T Q^T
      uint32_t hi[4], lo[4];
      split_a(S.s[2 * kb], S.s[2 * kb + 1], hi, lo);
      const uint32_t qa = st + (at.row_b * Sh::kRow + kb * 16 + at.col_b) * 2;
#pragma unroll
      for (int np = 0; np < 4; np += 2) {
        uint32_t b[4], d[4];
        const uint32_t q0 = qa + np * 16 * Sh::kRow * 2, q1 = q0 + 16 * Sh::kRow * 2;
        ldmatrix_x4(b, q0);
        ldmatrix_x4(d, q1);
        Mma::run(O[2 * np], hi, b[0], b[1]);
        Mma::run(O[2 * np + 1], hi, b[2], b[3]);
        Mma::run(O[2 * np + 2], hi, d[0], d[1]);
        Mma::run(O[2 * np + 3], hi, d[2], d[3]);
        Mma::run(O[2 * np], lo, b[0], b[1]);
        Mma::run(O[2 * np + 1], lo, b[2], b[3]);
        Mma::run(O[2 * np + 2], lo, d[0], d[1]);
        Mma::run(O[2 * np + 3], lo, d[2], d[3]);
        ldmatrix_x4(b, q0 + Sh::kVec);
        ldmatrix_x4(d, q1 + Sh::kVec);
        Mma::run(O[2 * np], hi, b[0], b[1]);
        Mma::run(O[2 * np + 1], hi, b[2], b[3]);
        Mma::run(O[2 * np + 2], hi, d[0], d[1]);
        Mma::run(O[2 * np + 3], hi, d[2], d[3]);
      }
    }
#pragma unroll
    for (int ib = 0; ib < 4; ++ib) mma_lower<false>(O, va[ib], va[ib], ad, ib, at);
#pragma unroll
    for (int n = 0; n < K / 8; ++n) {
      const float2 d = *reinterpret_cast<const float2*>(decay + n * 8 + c2);
      S.s[n][0] *= d.x; S.s[n][1] *= d.y; S.s[n][2] *= d.x; S.s[n][3] *= d.y;
    }
#pragma unroll
    for (int term = 0; term < 2; ++term)
#pragma unroll
      for (int ib = 0; ib < 4; ++ib) {
        const uint32_t ka = st + (2 + term) * Sh::kVec + ((ib * 16 + at.row_t) * Sh::kRow + at.col_t) * 2;
#pragma unroll
        for (int np = 0; np < K / 16; ++np) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, ka + np * 32);
          Mma::run(S.s[2 * np], va[ib], b[0], b[1]);
          Mma::run(S.s[2 * np + 1], va[ib], b[2], b[3]);
        }
      }
    const int64_t row0 = static_cast<int64_t>(first) + c * kChunk;
    store_out(O, reinterpret_cast<__nv_bfloat16*>(stage + 4 * Sh::kVec) + warp * 16, vrow,
              p.out + row0 * p.out_stride + static_cast<int64_t>(h) * p.V + p0 + warp * 16, p.out_stride,
              min(kChunk, n_tok - c * kChunk), pw - warp * 16, lane);
  }
  if (live && work) S.store(gS, p0 + warp * 16, p0 + pw, p.V, p.K, lane);
}

static int64_t gla_scratch_bytes(int K) {
  int64_t n = 0;
  chunk_dispatch(K, [&](auto kk) { n = GlaScratch<decltype(kk)::value>::kBytes; return 0; });
  return n;
}

}  // namespace mv

// Bytes of scratch for a step, or -1 when the kernels do not take the sizes.
extern "C" int64_t mv_gla_chunk_workspace_bytes(int64_t tokens, int num_seqs, int heads, int dim, int vdim) {
  using namespace mv;
  if (tokens < 0 || num_seqs < 0 || heads <= 0 || !chunk_takes(dim, vdim)) return -1;
  return chunk_bound(tokens, num_seqs) * heads * gla_scratch_bytes(dim);
}

// Both recurrences; kTime: p.zf, p.w0 and p.bonus, else p.z and p.inv_tau.
template <bool kTime>
static int run_chunks(const char* what, const mv::GlaChunkParams& p, int64_t tokens, int64_t workspace_bytes, cudaStream_t st) {
  using namespace mv;
  const int num_seqs = p.num_seqs, heads = p.heads, dim = p.K, vdim = p.V;
  if (num_seqs < 0 || tokens < 0 || heads <= 0 || heads > 65535 || !chunk_takes(dim, vdim))
    return fail(MV_ERR_SHAPE, "%s: heads %d, dim %d, vdim %d", what, heads, dim, vdim);
  if (num_seqs == 0 || tokens == 0) return MV_OK;
  if (!p.out || !p.q || !p.k || !p.v || !(kTime ? p.zf && p.w0 && p.bonus : p.z != nullptr) || !p.cu || !p.slots || !p.start || !p.state)
    return fail(MV_ERR_NULL, "%s: null pointer", what);
  if (!vec8_ok(p.out, p.out_stride, 2) || !vec8_ok(p.q, p.stride, 2) || !vec8_ok(p.k, p.stride, 2) || !vec8_ok(p.v, p.stride, 2))
    return fail(MV_ERR_ALIGN, "%s: rows must start on 16-byte boundaries", what);
  const int64_t chunks = chunk_bound(tokens, num_seqs);
  if (!p.scratch || !aligned16(p.scratch) || workspace_bytes < chunks * heads * gla_scratch_bytes(dim))
    return fail(MV_ERR_WORKSPACE, "%s: workspace", what);
  return chunk_dispatch(dim, [&](auto kk) {
    constexpr int K = decltype(kk)::value;
    constexpr int prep = GlaPrepShape<K>::kBytes;
    cudaError_t e = cudaFuncSetAttribute(gla_prepare_kernel<K, kTime>, cudaFuncAttributeMaxDynamicSharedMemorySize, prep);
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
    gla_prepare_kernel<K, kTime><<<dim3(static_cast<unsigned>(chunks), heads), kGpThreads, prep, st>>>(p);
    int rc = check_launch(what);
    if (rc) return rc;
    const int pb = chunk_columns(static_cast<int64_t>(num_seqs) * heads, vdim), smem = 2 * GlaChunkShape<K>::stage(pb);
    e = cudaFuncSetAttribute(gla_chunk_kernel<K>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
    gla_chunk_kernel<K><<<dim3(num_seqs, heads, (vdim + pb - 1) / pb), kChunkThreads, smem, st>>>(p, pb);
    return check_launch(what);
  });
}

extern "C" int mv_gla_chunk_scan(void* out, int64_t out_stride, const void* q, const void* k, const void* v, int64_t stride,
                                 const void* z, int64_t z_stride, float tau, const int32_t* cu, int num_seqs,
                                 int64_t tokens, const int32_t* slots, const int32_t* start, float* state, int num_slots,
                                 int heads, int dim, int vdim, float q_scale, void* workspace, int64_t workspace_bytes,
                                 void* stream) {
  using namespace mv;
  if (!(tau > 0.f)) return fail(MV_ERR_SHAPE, "gla_chunk_scan: tau %f", tau);
  auto c = [](const void* x) { return static_cast<const __nv_bfloat16*>(x); };
  const GlaChunkParams p{static_cast<__nv_bfloat16*>(out), out_stride, c(q), c(k), c(v), stride, c(z), z_stride, 1.f / tau, q_scale,
                         nullptr, nullptr, nullptr,
                         cu, slots, start, num_seqs, state, num_slots, heads, dim, vdim, static_cast<unsigned char*>(workspace)};
  return run_chunks<false>("gla_chunk_scan", p, tokens, workspace_bytes, static_cast<cudaStream_t>(stream));
}

extern "C" int mv_time_chunk_scan(void* out, int64_t out_stride, const void* r, const void* k, const void* v, int64_t stride,
                                  const float* z, int64_t z_stride, const void* w0, const void* bonus, const int32_t* cu,
                                  int num_seqs, int64_t tokens, const int32_t* slots, const int32_t* start, float* state,
                                  int num_slots, int heads, int dim, int vdim, void* workspace, int64_t workspace_bytes,
                                  void* stream) {
  using namespace mv;
  auto c = [](const void* x) { return static_cast<const __nv_bfloat16*>(x); };
  const GlaChunkParams p{static_cast<__nv_bfloat16*>(out), out_stride, c(r), c(k), c(v), stride, nullptr, z_stride, 1.f, 1.f,
                         z, c(w0), c(bonus),
                         cu, slots, start, num_seqs, state, num_slots, heads, dim, vdim, static_cast<unsigned char*>(workspace)};
  return run_chunks<true>("time_chunk_scan", p, tokens, workspace_bytes, static_cast<cudaStream_t>(stream));
}
