// Matrix memory with exponential gates (mLSTM) in chunks of 64 tokens.  With b_t the running sums of the forget gates' logarithms
// inside the chunk, m_0 the maximum in front of it, a_j = i_j - m_0 - b_j and M_t = m_t - m_0 - b_t, all of which the chain of
// mlstm.cu fixes, every power below is at most one:
//   O = alpha (Q S_0) + A V,     A[t, j] = q_t k_j e^(a_j - M_t), j <= t,     alpha_t = e^(-M_t)
//   S = e^(-M_last) S_0 + (w K)^T V,     w_j = e^(a_j - M_last);     n the same with V = 1
//   denominator of t = max(|alpha_t q_t n_0 + sum_j A[t, j]|, e^-m_t) + 1e-6
// mlstm_prepare_kernel  per chunk and head: the factors, A in two terms, its row sums, sum_j w_j k_j
// mlstm_chunk_kernel    per sequence, head and block of value columns: see state_chunk.cuh.  The first block of columns also
//                       carries n and writes the denominators.
// Q, K and V enter as the projection left them, their factors as fp32 on accumulators or, w, on V^T in two terms.
#include "state_chunk.cuh"

namespace mv {

constexpr int kMpThreads = 256;

struct MemChunkParams {
  __nv_bfloat16* out; int64_t out_stride;
  float* den;
  const __nv_bfloat16 *q, *k, *v; int64_t stride;
  const float4* chain;                          // (tokens, heads) i, f, m before, m after
  float q_scale;
  const int32_t *cu, *slots, *start;
  int num_seqs;
  float *state, *n_state; int num_slots, heads, K, V;
  unsigned char* scratch;                       // [chunk][head][A hi, A lo, vectors]
};

// Vectors of a chunk and head, in floats.
template <int K> struct MemVec {
  static constexpr int kAlpha = 0, kWrite = kChunk, kRow = 2 * kChunk, kFloor = 3 * kChunk, kSum = 4 * kChunk, kDecay = kSum + K,
                       kCount = kDecay + 4;
  static constexpr int64_t kA = 2 * kChunk * kChunk * 2, kBytes = kA + kCount * 4;
};

template <int K>
__global__ void __launch_bounds__(kMpThreads) mlstm_prepare_kernel(const MemChunkParams p) {
  using Vc = MemVec<K>;
  constexpr int ROW = K + 8;
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16 *sQ = reinterpret_cast<__nv_bfloat16*>(smem), *sK = sQ + kChunk * ROW;
  __shared__ float s_a[kChunk], s_M[kChunk], s_w[kChunk], s_part[4][kChunk];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y;
  int seq, chunk;
  if (!find_chunk(p.cu, p.num_seqs, blockIdx.x, seq, chunk)) return;     // uniform: the grid is an upper bound
  const int64_t first = p.cu[seq] + static_cast<int64_t>(chunk) * kChunk;
  const int nt = min(kChunk, static_cast<int>(p.cu[seq + 1] - first));
  unsigned char* dst = p.scratch + (static_cast<int64_t>(blockIdx.x) * p.heads + h) * Vc::kBytes;
  float* vec = reinterpret_cast<float*>(dst + Vc::kA);
  {
    const uint32_t qd = smem_u32(sQ), kd = smem_u32(sK);
    for (int i = tid; i < kChunk * (K / 8); i += kMpThreads) {
      const int r = i / (K / 8), c = (i % (K / 8)) * 8;
      const bool ok = r < nt && c < p.K;
      const int64_t off = ok ? (first + r) * p.stride + h * p.K + c : 0;
      cp_async16(qd + (r * ROW + c) * 2, p.q + off, ok ? 16 : 0);
      cp_async16(kd + (r * ROW + c) * 2, p.k + off, ok ? 16 : 0);
    }
    cp_async_commit();
  }
  if (warp == 0) {                       // two neighbouring tokens per lane, base-2 logarithms
    float b[2], m[2], a[2], M[2], run = 0.f;
    const float m0 = p.chain[first * p.heads + h].z;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = lane * 2 + e;
      const float4 c = t < nt ? p.chain[(first + t) * p.heads + h] : make_float4(0.f, 0.f, 0.f, 0.f);
      run += c.y * kLog2e;
      b[e] = run;
      a[e] = (c.x - m0) * kLog2e;
      m[e] = c.w;
    }
    float before = run;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, before, o);
      if (lane >= o) before += v;
    }
    before -= run;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      a[e] -= before + b[e];
      M[e] = (m[e] - m0) * kLog2e - (before + b[e]);
    }
    const float last = __shfl_sync(0xffffffffu, (nt - 1) & 1 ? M[1] : M[0], (nt - 1) >> 1);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = lane * 2 + e;
      const bool on = t < nt;
      s_a[t] = on ? a[e] : 0.f;
      s_M[t] = on ? M[e] : 1e30f;          // rows past the end become zero
      s_w[t] = on ? fast_exp2(a[e] - last) : 0.f;
      vec[Vc::kWrite + t] = s_w[t];
      vec[Vc::kAlpha + t] = on ? p.q_scale * fast_exp2(-M[e]) : 0.f;
      vec[Vc::kFloor + t] = on ? fast_exp2(-m[e] * kLog2e) : 1.f;
    }
    if (lane == 0) vec[Vc::kDecay] = fast_exp2(-last);
  }
  cp_async_wait<0>();
  __syncthreads();
  const LaneAt at(lane);
  uint32_t* gA = reinterpret_cast<uint32_t*>(dst);
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  // blocks 0 .. 5 below the diagonal, (1,0) (2,0) (2,1) (3,0) (3,1) (3,2), then the four on it
#pragma unroll 1
  for (int blk = warp; blk < 10; blk += kMpThreads / 32) {
    const bool diag = blk >= 6;
    const int bi = diag ? blk - 6 : blk == 0 ? 1 : blk < 3 ? 2 : 3, bj = diag ? bi : blk - bi * (bi - 1) / 2;
    const uint32_t qa = smem_u32(sQ) + ((bi * 16 + at.row_t) * ROW + at.col_t) * 2;
    const uint32_t kb = smem_u32(sK) + ((bj * 16 + at.row_b) * ROW + at.col_b) * 2;
    float acc[2][4] = {};
#pragma unroll
    for (int c = 0; c < K; c += 16) {
      uint32_t a[4], b[4];
      ldmatrix_x4(a, qa + c * 2);
      ldmatrix_x4(b, kb + c * 2);
      Mma::run(acc[0], a, b[0], b[1]);
      Mma::run(acc[1], a, b[2], b[3]);
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = bi * 16 + g + half * 8;
      const float M = s_M[t];
      float sum = 0.f;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int j = bj * 16 + n * 8 + c2;
        const float x = j <= t ? acc[n][2 * half] * p.q_scale * fast_exp2(s_a[j] - M) : 0.f;
        const float y = j + 1 <= t ? acc[n][2 * half + 1] * p.q_scale * fast_exp2(s_a[j + 1] - M) : 0.f;
        sum += x + y;
        uint32_t hi, lo;
        split2(x, y, hi, lo);
        gA[(t * kChunk + j) / 2] = hi;
        gA[kChunk * kChunk / 2 + (t * kChunk + j) / 2] = lo;
      }
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      if ((lane & 3) == 0) s_part[bj][t] = sum;
    }
  }
  for (int c = tid; c < K; c += kMpThreads) {
    float s[4] = {};
#pragma unroll 4
    for (int j = 0; j < kChunk; j += 4)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[e] = fmaf(s_w[j + e], __bfloat162float(sK[(j + e) * ROW + c]), s[e]);
    vec[Vc::kSum + c] = (s[0] + s[1]) + (s[2] + s[3]);
  }
  __syncthreads();
  for (int t = tid; t < kChunk; t += kMpThreads) {
    float s = 0.f;
    for (int bj = 0; bj <= t / 16; ++bj) s += s_part[bj][t];
    vec[Vc::kRow + t] = s;
  }
}

template <int K> struct MemChunkShape {
  static constexpr int kRow = K + 8;
  static constexpr int kVec = kChunk * kRow * 2, kTile = 2 * kChunk * kCkRow * 2;       // bytes
  static constexpr int v_bytes(int pb) { return kChunk * (pb + 8) * 2; }
  static constexpr int stage(int pb) { return 2 * kVec + v_bytes(pb) + kTile + MemVec<K>::kCount * 4; }
};

template <int K>
__global__ void __launch_bounds__(kChunkThreads, 1) mlstm_chunk_kernel(const MemChunkParams p, int pb) {
  using Sh = MemChunkShape<K>;
  using Vc = MemVec<K>;
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float s_n[2][K];
  const int s = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * pb, pw = min(pb, p.V - p0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c2 = (lane & 3) * 2;
  const int vrow = pb + 8;
  const int first = p.cu[s], n_tok = p.cu[s + 1] - first;
  if (n_tok <= 0) return;
  const int chunk0 = chunks_before(p.cu, s), chunks = (n_tok + kChunk - 1) / kChunk;
  const int slot = p.slots[s], st0 = p.start[s];
  const bool live = slot >= 0 && slot < p.num_slots && st0 >= 0, keeps_n = blockIdx.z == 0;
  float* gS = p.state + (static_cast<int64_t>(live ? slot : 0) * p.heads + h) * p.K * p.V;
  float* gN = p.n_state + (static_cast<int64_t>(live ? slot : 0) * p.heads + h) * p.K;
  const int stage_bytes = Sh::stage(pb);
  const uint32_t base = smem_u32(smem);
  const __nv_bfloat16* v = p.v + static_cast<int64_t>(h) * p.V + p0;

  auto issue = [&](int c) {
    const uint32_t st = base + (c & 1) * stage_bytes;
    const int64_t row0 = static_cast<int64_t>(first) + c * kChunk;
    const int nt = min(kChunk, n_tok - c * kChunk);
    const unsigned char* src = p.scratch + (static_cast<int64_t>(chunk0 + c) * p.heads + h) * Vc::kBytes;
    for (int i = tid; i < kChunk * (K / 8); i += kChunkThreads) {
      const int r = i / (K / 8), cc = (i % (K / 8)) * 8;
      const bool ok = r < nt && cc < p.K;
      const int64_t off = ok ? (row0 + r) * p.stride + h * p.K + cc : 0;
      cp_async16(st + (r * Sh::kRow + cc) * 2, p.q + off, ok ? 16 : 0);
      cp_async16(st + Sh::kVec + (r * Sh::kRow + cc) * 2, p.k + off, ok ? 16 : 0);
    }
    const uint32_t vd = st + 2 * Sh::kVec, ad = vd + Sh::v_bytes(pb);
    for (int i = tid; i < kChunk * (pb / 8); i += kChunkThreads) {
      const int r = i / (pb / 8), cc = (i % (pb / 8)) * 8;
      const bool ok = r < nt && cc < pw;
      cp_async16(vd + (r * vrow + cc) * 2, ok ? v + (row0 + r) * p.stride + cc : p.v, ok ? 16 : 0);
    }
    load_lower(ad, reinterpret_cast<const __nv_bfloat16*>(src), tid, kChunkThreads);
    for (int i = tid; i < Vc::kCount / 4; i += kChunkThreads) cp_async16(ad + Sh::kTile + i * 16, src + Vc::kA + i * 16, 16);
    cp_async_commit();
  };
  issue(0);
  const bool work = warp * 16 < pw;
  ChunkState<K> S;
  S.load(gS, p0 + warp * 16, p0 + pw, p.V, p.K, lane, work && live && st0 > 0);
  for (int i = tid; i < K; i += kChunkThreads) s_n[0][i] = keeps_n && live && st0 > 0 && i < p.K ? gN[i] : 0.f;
  const LaneAt at(lane);
  for (int c = 0; c < chunks; ++c) {
    cp_async_wait<0>();
    __syncthreads();                     // chunk c is here, and nobody reads the other stage any more
    if (c + 1 < chunks) issue(c + 1);
    unsigned char* stage = smem + (c & 1) * stage_bytes;
    const uint32_t st = base + (c & 1) * stage_bytes;
    const uint32_t kd = st + Sh::kVec, vd = st + 2 * Sh::kVec, ad = vd + Sh::v_bytes(pb);
    const float* vec = reinterpret_cast<const float*>(stage + 2 * Sh::kVec + Sh::v_bytes(pb) + Sh::kTile);
    const int nt = min(kChunk, n_tok - c * kChunk);
    if (keeps_n) {
      const __nv_bfloat16* sQ = reinterpret_cast<const __nv_bfloat16*>(stage);
      const float* n_old = s_n[c & 1];
      constexpr int kPer = kChunk / (kChunkThreads / 32);
      float dot[kPer];
#pragma unroll
      for (int r = 0; r < kPer; ++r) {
        dot[r] = 0.f;
#pragma unroll
        for (int m = 0; m < K / 32; ++m)
          dot[r] = fmaf(n_old[m * 32 + lane], __bfloat162float(sQ[(warp * kPer + r) * Sh::kRow + m * 32 + lane]), dot[r]);
      }
#pragma unroll
      for (int r = 0; r < kPer; ++r) {
        dot[r] = warp_sum(dot[r]);
        const int t = warp * kPer + r;
        if (lane == 0 && t < nt)
          p.den[(static_cast<int64_t>(first) + c * kChunk + t) * p.heads + h] =
              fmaxf(fabsf(fmaf(vec[Vc::kAlpha + t], dot[r], vec[Vc::kRow + t])), vec[Vc::kFloor + t]) + kMemFloor;
      }
      // read by everybody behind the next chunk's barrier
      for (int i = tid; i < K; i += kChunkThreads) s_n[(c + 1) & 1][i] = fmaf(vec[Vc::kDecay], n_old[i], vec[Vc::kSum + i]);
    }
    if (!work) continue;
    uint32_t va[4][4];                   // V^T, an A operand
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
        ldmatrix_x4(b, qa + np * 16 * Sh::kRow * 2);
        ldmatrix_x4(d, qa + (np + 1) * 16 * Sh::kRow * 2);
        Mma::run(O[2 * np], hi, b[0], b[1]);
        Mma::run(O[2 * np + 1], hi, b[2], b[3]);
        Mma::run(O[2 * np + 2], hi, d[0], d[1]);
        Mma::run(O[2 * np + 3], hi, d[2], d[3]);
        Mma::run(O[2 * np], lo, b[0], b[1]);
        Mma::run(O[2 * np + 1], lo, b[2], b[3]);
        Mma::run(O[2 * np + 2], lo, d[0], d[1]);
        Mma::run(O[2 * np + 3], lo, d[2], d[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const float2 a = *reinterpret_cast<const float2*>(vec + Vc::kAlpha + n * 8 + c2);
      O[n][0] *= a.x; O[n][1] *= a.y; O[n][2] *= a.x; O[n][3] *= a.y;
    }
#pragma unroll
    for (int ib = 0; ib < 4; ++ib) mma_lower<false>(O, va[ib], va[ib], ad, ib, at);
    const float decay = vec[Vc::kDecay];
#pragma unroll
    for (int n = 0; n < K / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) S.s[n][e] *= decay;
#pragma unroll
    for (int ib = 0; ib < 4; ++ib) {
      uint32_t hi[4], lo[4];             // (w V)^T
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float2 w = *reinterpret_cast<const float2*>(vec + Vc::kWrite + ib * 16 + (x >> 1) * 8 + c2);
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&va[ib][x]));
        split2(f.x * w.x, f.y * w.y, hi[x], lo[x]);
      }
      const uint32_t ka = kd + ((ib * 16 + at.row_t) * Sh::kRow + at.col_t) * 2;
#pragma unroll
      for (int np = 0; np < K / 16; np += 2) {
        uint32_t b[4], d[4];
        ldmatrix_x4_trans(b, ka + np * 32);
        ldmatrix_x4_trans(d, ka + (np + 1) * 32);
        Mma::run(S.s[2 * np], hi, b[0], b[1]);
        Mma::run(S.s[2 * np + 1], hi, b[2], b[3]);
        Mma::run(S.s[2 * np + 2], hi, d[0], d[1]);
        Mma::run(S.s[2 * np + 3], hi, d[2], d[3]);
        Mma::run(S.s[2 * np], lo, b[0], b[1]);
        Mma::run(S.s[2 * np + 1], lo, b[2], b[3]);
        Mma::run(S.s[2 * np + 2], lo, d[0], d[1]);
        Mma::run(S.s[2 * np + 3], lo, d[2], d[3]);
      }
    }
    const int64_t row0 = static_cast<int64_t>(first) + c * kChunk;
    store_out(O, reinterpret_cast<__nv_bfloat16*>(stage + 2 * Sh::kVec) + warp * 16, vrow,
              p.out + row0 * p.out_stride + static_cast<int64_t>(h) * p.V + p0 + warp * 16, p.out_stride, nt, pw - warp * 16, lane);
  }
  if (live && work) S.store(gS, p0 + warp * 16, p0 + pw, p.V, p.K, lane);
  if (live && keeps_n)
    for (int i = tid; i < p.K; i += kChunkThreads) gN[i] = s_n[chunks & 1][i];      // written by this thread
}

static int64_t mlstm_scratch_bytes(int K) {
  int64_t n = 0;
  chunk_dispatch(K, [&](auto kk) { n = MemVec<decltype(kk)::value>::kBytes; return 0; });
  return n;
}

}  // namespace mv

// Bytes of scratch for a step, or -1 when the kernels do not take the sizes.
extern "C" int64_t mv_mlstm_chunk_workspace_bytes(int64_t tokens, int num_seqs, int heads, int dim, int vdim) {
  using namespace mv;
  if (tokens < 0 || num_seqs < 0 || heads <= 0 || !chunk_takes(dim, vdim)) return -1;
  return chunk_bound(tokens, num_seqs) * heads * mlstm_scratch_bytes(dim);
}

extern "C" int mv_mlstm_chunk_scan(void* out, int64_t out_stride, float* den, const void* q, const void* k, const void* v,
                                   int64_t stride, const float* chain, const int32_t* cu, int num_seqs, int64_t tokens,
                                   const int32_t* slots, const int32_t* start, float* S, float* n, int num_slots, int heads,
                                   int dim, int vdim, float q_scale, void* workspace, int64_t workspace_bytes, void* stream) {
  using namespace mv;
  if (num_seqs < 0 || tokens < 0 || heads <= 0 || heads > 65535 || !chunk_takes(dim, vdim))
    return fail(MV_ERR_SHAPE, "mlstm_chunk_scan: heads %d, dim %d, vdim %d", heads, dim, vdim);
  if (num_seqs == 0 || tokens == 0) return MV_OK;
  if (!out || !den || !q || !k || !v || !chain || !cu || !slots || !start || !S || !n) return fail(MV_ERR_NULL, "mlstm_chunk_scan: null pointer");
  if (!vec8_ok(out, out_stride, 2) || !vec8_ok(q, stride, 2) || !vec8_ok(k, stride, 2) || !vec8_ok(v, stride, 2) || !aligned16(chain))
    return fail(MV_ERR_ALIGN, "mlstm_chunk_scan: rows must start on 16-byte boundaries");
  const int64_t chunks = chunk_bound(tokens, num_seqs);
  if (!workspace || !aligned16(workspace) || workspace_bytes < chunks * heads * mlstm_scratch_bytes(dim))
    return fail(MV_ERR_WORKSPACE, "mlstm_chunk_scan: workspace");
  auto c = [](const void* x) { return static_cast<const __nv_bfloat16*>(x); };
  const MemChunkParams p{static_cast<__nv_bfloat16*>(out), out_stride, den, c(q), c(k), c(v), stride, reinterpret_cast<const float4*>(chain),
                         q_scale, cu, slots, start, num_seqs, S, n, num_slots, heads, dim, vdim, static_cast<unsigned char*>(workspace)};
  auto st = static_cast<cudaStream_t>(stream);
  return chunk_dispatch(dim, [&](auto kk) {
    constexpr int K = decltype(kk)::value;
    constexpr int prep = 2 * kChunk * (K + 8) * 2;
    mlstm_prepare_kernel<K><<<dim3(static_cast<unsigned>(chunks), heads), kMpThreads, prep, st>>>(p);
    int rc = check_launch("mlstm_prepare");
    if (rc) return rc;
    const int pb = chunk_columns(static_cast<int64_t>(num_seqs) * heads, vdim), smem = 2 * MemChunkShape<K>::stage(pb);
    const cudaError_t e = cudaFuncSetAttribute(mlstm_chunk_kernel<K>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "mlstm_chunk_scan: %s", cudaGetErrorString(e));
    mlstm_chunk_kernel<K><<<dim3(num_seqs, heads, (vdim + pb - 1) / pb), kChunkThreads, smem, st>>>(p, pb);
    return check_launch("mlstm_chunk");
  });
}
