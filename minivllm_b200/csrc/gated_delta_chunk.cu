// The gated delta rule in chunks of 64 tokens.  With c_t the running sum of the log2 decays inside the chunk, k and q the
// unscaled rows, kappa_t and chi_t the factors that make them unit vectors (chi with the scale of q):
//   (I + A) U = beta V - beta 2^c kappa (K S_0),    A[t, i] = beta_t 2^(c_t - c_i) kappa_t kappa_i (k_t . k_i), i < t
//   O = 2^c chi (Q S_0) + M U,                      M[t, i] = 2^(c_t - c_i) chi_t kappa_i (q_t . k_i),        i <= t
//   S = 2^c_last S_0 + K^T (2^(c_last - c) kappa U)
// delta_prepare_kernel  per chunk and KV head: the products K K^T and Q K^T, and per head T = (I + A)^-1 by forward
//                       substitution in fp32 (a thread per column), M, and the factors per token
// delta_chunk_kernel    per sequence, head and block of value columns: see state_chunk.cuh
// K and Q enter as the convolution left them; T, M, U and S in two terms.
#include "state_chunk.cuh"

namespace mv {

constexpr int kDpThreads = 128;
constexpr int kDcPar = 4 * kChunk + 4;          // floats per chunk and head: beta, beta 2^c kappa, 2^c chi, 2^(last - c) kappa; 2^c_last
constexpr int64_t kDcTile = 2 * kChunk * kChunk;        // elements of a tile in two terms
constexpr int64_t kDcBytes = 2 * kDcTile * 2 + (kDcPar * 4 + 15) / 16 * 16;     // scratch per chunk and head

struct DeltaChunkParams {
  __nv_bfloat16* out; int64_t out_stride;
  const __nv_bfloat16* qkv; int64_t stride;
  const __nv_bfloat16 *beta, *a; int64_t ba_stride;
  const __nv_bfloat16 *A_log, *dt_bias;
  const int32_t *cu, *slots, *start;
  int num_seqs;
  float* state; int num_slots, heads, kv_heads, K, V;
  float q_scale;
  unsigned char* scratch;                       // [chunk][head][T hi, T lo, M hi, M lo, factors]
};

__device__ __forceinline__ unsigned char* delta_scratch(const DeltaChunkParams& p, int64_t chunk, int h) {
  return p.scratch + (chunk * p.heads + h) * kDcBytes;
}

template <int K> struct DeltaPrepShape {
  static constexpr int kRow = K + 8, kA = 68, kT = 65;
  static constexpr int kTiles = 2 * kChunk * kRow * 2, kMats = kChunk * (kA + kT) * 4;
  static constexpr int kBytes = kTiles > kMats ? kTiles : kMats;      // the matrices lie over the tiles of K and Q
};

template <int K>
__global__ void __launch_bounds__(kDpThreads, 4) delta_prepare_kernel(const DeltaChunkParams p) {
  using Sh = DeltaPrepShape<K>;
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16 *sK = reinterpret_cast<__nv_bfloat16*>(smem), *sQ = sK + kChunk * Sh::kRow;
  float *sA = reinterpret_cast<float*>(smem), *sT = sA + kChunk * Sh::kA;      // A by column, T by row
  __shared__ float s_ks[kChunk], s_qs[kChunk], s_c[kChunk], s_b[kChunk];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kh = blockIdx.y;
  int seq, chunk;
  if (!find_chunk(p.cu, p.num_seqs, blockIdx.x, seq, chunk)) return;     // uniform: the grid is an upper bound
  const int64_t first = p.cu[seq] + static_cast<int64_t>(chunk) * kChunk;
  const int nt = min(kChunk, static_cast<int>(p.cu[seq + 1] - first));
  {
    const __nv_bfloat16 *q = p.qkv + kh * p.K, *k = q + p.kv_heads * p.K;
    const uint32_t kd = smem_u32(sK), qd = smem_u32(sQ);
    for (int i = tid; i < kChunk * (K / 8); i += kDpThreads) {
      const int r = i / (K / 8), c = (i % (K / 8)) * 8;
      const bool ok = r < nt && c < p.K;
      const int64_t off = ok ? (first + r) * p.stride + c : 0;
      cp_async16(kd + (r * Sh::kRow + c) * 2, k + off, ok ? 16 : 0);
      cp_async16(qd + (r * Sh::kRow + c) * 2, q + off, ok ? 16 : 0);
    }
    cp_async_commit();
    cp_async_wait<0>();
  }
  __syncthreads();
  for (int r = warp; r < kChunk; r += kDpThreads / 32) {
    float kk = 0.f, qq = 0.f;
#pragma unroll
    for (int m = 0; m < K / 32; ++m) {
      const float a = __bfloat162float(sK[r * Sh::kRow + m * 32 + lane]), b = __bfloat162float(sQ[r * Sh::kRow + m * 32 + lane]);
      kk = fmaf(a, a, kk);
      qq = fmaf(b, b, qq);
    }
    kk = warp_sum(kk);
    qq = warp_sum(qq);
    if (lane == 0) {
      s_ks[r] = 1.f / sqrtf(kk + kUnitEps);
      s_qs[r] = p.q_scale / sqrtf(qq + kUnitEps);
    }
  }
  const LaneAt at(lane);
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  float kk[8][4] = {}, qk[8][4] = {};
  {
    // A operands: rows 16 warp .. + 15
    const uint32_t ka = smem_u32(sK) + ((warp * 16 + at.row_t) * Sh::kRow + at.col_t) * 2, qa = ka + kChunk * Sh::kRow * 2;
    const uint32_t kb = smem_u32(sK) + (at.row_b * Sh::kRow + at.col_b) * 2;
#pragma unroll
    for (int i = 0; i < K; i += 16) {
      uint32_t x[4], y[4], b[4];
      ldmatrix_x4(x, ka + i * 2);
      ldmatrix_x4(y, qa + i * 2);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        if (np > warp) continue;
        ldmatrix_x4(b, kb + (np * 16 * Sh::kRow + i) * 2);
        Mma::run(kk[2 * np], x, b[0], b[1]);
        Mma::run(kk[2 * np + 1], x, b[2], b[3]);
        Mma::run(qk[2 * np], y, b[0], b[1]);
        Mma::run(qk[2 * np + 1], y, b[2], b[3]);
      }
    }
  }
  __syncthreads();
  const int group = p.heads / p.kv_heads;
  for (int hg = 0; hg < group; ++hg) {
    const int h = kh * group + hg;
    unsigned char* dst = delta_scratch(p, blockIdx.x, h);
    uint32_t* gT = reinterpret_cast<uint32_t*>(dst);                       // pairs of elements
    uint32_t* gM = gT + kDcTile / 2;
    if (warp == 0) {
      float* par = reinterpret_cast<float*>(gM + kDcTile / 2);
      const float A_log = __bfloat162float(p.A_log[h]), dt_bias = __bfloat162float(p.dt_bias[h]);
      float l[2], b[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = lane * 2 + i;
        const bool ok = t < nt;
        const int64_t row = (first + t) * p.ba_stride + h;
        l[i] = ok ? head_log_decay(__bfloat162float(p.a[row]), A_log, dt_bias) * kLog2e : 0.f;
        b[i] = ok ? sigmoid_f(__bfloat162float(p.beta[row])) : 0.f;        // tokens past the end change nothing
      }
      float run = l[0] + l[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += v;
      }
      const float last = __shfl_sync(0xffffffffu, run, 31);
      const float c[2] = {run - l[1], run};
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = lane * 2 + i;
        const float e = fast_exp2(c[i]);
        s_c[t] = c[i];
        s_b[t] = b[i];
        par[t] = b[i];
        par[kChunk + t] = b[i] * e * s_ks[t];
        par[2 * kChunk + t] = e * s_qs[t];
        par[3 * kChunk + t] = fast_exp2(last - c[i]) * s_ks[t];
      }
      if (lane == 0) par[4 * kChunk] = fast_exp2(last);
    }
    __syncthreads();
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      if (n > 2 * warp + 1) continue;
      const int i0 = n * 8 + c2;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = warp * 16 + g + half * 8;
        const float ct = s_c[t], bk = s_b[t] * s_ks[t], qs = s_qs[t];
        float m[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = i0 + e;
          const float d = i <= t ? fast_exp2(ct - s_c[i]) * s_ks[i] : 0.f;
          m[e] = qs * d * qk[n][2 * half + e];
          sA[i * Sh::kA + t] = i < t ? bk * d * kk[n][2 * half + e] : 0.f;
        }
        uint32_t hi, lo;
        split2(m[0], m[1], hi, lo);
        gM[(t * kChunk + i0) / 2] = hi;
        gM[kChunk * kChunk / 2 + (t * kChunk + i0) / 2] = lo;
      }
    }
    __syncthreads();
    if (tid < kChunk) {        // column tid of the inverse
#pragma unroll 1
      for (int rb = tid / 16; rb < 4; ++rb) {
        float x[16];
#pragma unroll
        for (int r = 0; r < 16; ++r) x[r] = rb * 16 + r == tid ? 1.f : 0.f;
#pragma unroll 2
        for (int i = tid / 16 * 16; i < rb * 16; ++i) {
          const float y = -sT[i * Sh::kT + tid];
          const float4* a4 = reinterpret_cast<const float4*>(sA + i * Sh::kA + rb * 16);
#pragma unroll
          for (int r4 = 0; r4 < 4; ++r4) {
            const float4 a = a4[r4];
            x[4 * r4] = fmaf(a.x, y, x[4 * r4]);
            x[4 * r4 + 1] = fmaf(a.y, y, x[4 * r4 + 1]);
            x[4 * r4 + 2] = fmaf(a.z, y, x[4 * r4 + 2]);
            x[4 * r4 + 3] = fmaf(a.w, y, x[4 * r4 + 3]);
          }
        }
#pragma unroll
        for (int i = 0; i < 15; ++i) {
          const float* a = sA + (rb * 16 + i) * Sh::kA + rb * 16;
#pragma unroll
          for (int r = i + 1; r < 16; ++r) x[r] = fmaf(-a[r], x[i], x[r]);
        }
#pragma unroll
        for (int r = 0; r < 16; ++r) sT[(rb * 16 + r) * Sh::kT + tid] = x[r];
      }
    }
    __syncthreads();
    for (int i = tid; i < kChunk * kChunk / 2; i += kDpThreads) {
      const int t = i / 32, j = (i % 32) * 2;
      if (j / 16 > t / 16) continue;
      uint32_t hi, lo;
      split2(sT[t * Sh::kT + j], sT[t * Sh::kT + j + 1], hi, lo);
      gT[i] = hi;
      gT[kChunk * kChunk / 2 + i] = lo;
    }
  }
}

template <int K> struct DeltaChunkShape {
  static constexpr int kRow = K + 8;
  static constexpr int kK = kChunk * kRow * 2, kTile = 2 * kChunk * kCkRow * 2, kParBytes = kDcPar * 4;
  static constexpr int stage(int pb) { return 2 * kK + kChunk * (pb + 8) * 2 + 2 * kTile + (kParBytes + 15) / 16 * 16; }
};

template <int K>
__global__ void __launch_bounds__(kChunkThreads, 1) delta_chunk_kernel(const DeltaChunkParams p, int pb) {
  using Sh = DeltaChunkShape<K>;
  extern __shared__ __align__(16) unsigned char smem[];
  const int s = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * pb, pw = min(pb, p.V - p0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c2 = (lane & 3) * 2;
  const int kh = h / (p.heads / p.kv_heads), vrow = pb + 8;
  const int first = p.cu[s], n_tok = p.cu[s + 1] - first;
  if (n_tok <= 0) return;
  const int chunk0 = chunks_before(p.cu, s), chunks = (n_tok + kChunk - 1) / kChunk;
  const int slot = p.slots[s], st0 = p.start[s];
  const bool live = slot >= 0 && slot < p.num_slots && st0 >= 0;
  float* gS = p.state + (static_cast<int64_t>(live ? slot : 0) * p.heads + h) * p.K * p.V;
  const int stage_bytes = Sh::stage(pb);
  const uint32_t base = smem_u32(smem);
  const __nv_bfloat16 *q = p.qkv + kh * p.K, *k = q + p.kv_heads * p.K;
  const __nv_bfloat16* v = p.qkv + 2 * p.kv_heads * p.K + static_cast<int64_t>(h) * p.V + p0;

  auto issue = [&](int c) {
    const uint32_t st = base + (c & 1) * stage_bytes;
    const int64_t row0 = static_cast<int64_t>(first) + c * kChunk;
    const int nt = min(kChunk, n_tok - c * kChunk);
    for (int i = tid; i < kChunk * (K / 8); i += kChunkThreads) {
      const int r = i / (K / 8), cc = (i % (K / 8)) * 8;
      const bool ok = r < nt && cc < p.K;
      const int64_t off = ok ? (row0 + r) * p.stride + cc : 0;
      cp_async16(st + (r * Sh::kRow + cc) * 2, k + off, ok ? 16 : 0);
      cp_async16(st + Sh::kK + (r * Sh::kRow + cc) * 2, q + off, ok ? 16 : 0);
    }
    const uint32_t vd = st + 2 * Sh::kK;
    for (int i = tid; i < kChunk * (pb / 8); i += kChunkThreads) {
      const int r = i / (pb / 8), cc = (i % (pb / 8)) * 8;
      const bool ok = r < nt && cc < pw;
      cp_async16(vd + (r * vrow + cc) * 2, ok ? v + (row0 + r) * p.stride + cc : v, ok ? 16 : 0);
    }
    const unsigned char* src = delta_scratch(p, chunk0 + c, h);
    const uint32_t td = vd + kChunk * vrow * 2;
    load_lower(td, reinterpret_cast<const __nv_bfloat16*>(src), tid, kChunkThreads);
    load_lower(td + Sh::kTile, reinterpret_cast<const __nv_bfloat16*>(src) + kDcTile, tid, kChunkThreads);
    for (int i = tid; i < kDcPar / 4; i += kChunkThreads) cp_async16(td + 2 * Sh::kTile + i * 16, src + 2 * kDcTile * 2 + i * 16, 16);
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
    const uint32_t vd = st + 2 * Sh::kK, td = vd + kChunk * vrow * 2, md = td + Sh::kTile;
    const float* par = reinterpret_cast<const float*>(stage + 2 * Sh::kK + kChunk * vrow * 2 + 2 * Sh::kTile);
    float P[8][4] = {}, O[8][4] = {};
#pragma unroll
    for (int kb = 0; kb < K / 16; ++kb) {        // S_0^T K^T and S_0^T Q^T
      uint32_t hi[4], lo[4];
      split_a(S.s[2 * kb], S.s[2 * kb + 1], hi, lo);
      const uint32_t ka = st + (at.row_b * Sh::kRow + kb * 16 + at.col_b) * 2;
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t b[4], d[4];
        ldmatrix_x4(b, ka + np * 16 * Sh::kRow * 2);
        ldmatrix_x4(d, ka + Sh::kK + np * 16 * Sh::kRow * 2);
        Mma::run(P[2 * np], hi, b[0], b[1]);
        Mma::run(P[2 * np + 1], hi, b[2], b[3]);
        Mma::run(O[2 * np], hi, d[0], d[1]);
        Mma::run(O[2 * np + 1], hi, d[2], d[3]);
        Mma::run(P[2 * np], lo, b[0], b[1]);
        Mma::run(P[2 * np + 1], lo, b[2], b[3]);
        Mma::run(O[2 * np], lo, d[0], d[1]);
        Mma::run(O[2 * np + 1], lo, d[2], d[3]);
      }
    }
#pragma unroll
    for (int np = 0; np < 4; ++np) {             // right-hand sides; O's factors
      uint32_t x[4];
      ldmatrix_x4_trans(x, vd + ((np * 16 + at.row_b) * vrow + warp * 16 + at.col_b) * 2);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int n = 2 * np + j, t = n * 8 + c2;
        const float2 b = *reinterpret_cast<const float2*>(par + t), bg = *reinterpret_cast<const float2*>(par + kChunk + t);
        const float2 f = *reinterpret_cast<const float2*>(par + 2 * kChunk + t);
        const float2 v0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x[2 * j]));
        const float2 v1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x[2 * j + 1]));
        P[n][0] = fmaf(-bg.x, P[n][0], b.x * v0.x);
        P[n][1] = fmaf(-bg.y, P[n][1], b.y * v0.y);
        P[n][2] = fmaf(-bg.x, P[n][2], b.x * v1.x);
        P[n][3] = fmaf(-bg.y, P[n][3], b.y * v1.y);
        O[n][0] *= f.x; O[n][1] *= f.y; O[n][2] *= f.x; O[n][3] *= f.y;
      }
    }
    float U[8][4] = {};
#pragma unroll
    for (int ib = 0; ib < 4; ++ib) {
      uint32_t hi[4], lo[4];
      split_a(P[2 * ib], P[2 * ib + 1], hi, lo);
      mma_lower<true>(U, hi, lo, td, ib, at);
    }
#pragma unroll
    for (int ib = 0; ib < 4; ++ib) {
      uint32_t hi[4], lo[4];
      split_a(U[2 * ib], U[2 * ib + 1], hi, lo);
      mma_lower<true>(O, hi, lo, md, ib, at);
    }
    const float last = par[4 * kChunk];
#pragma unroll
    for (int n = 0; n < K / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) S.s[n][e] *= last;
#pragma unroll
    for (int ib = 0; ib < 4; ++ib) {
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const float2 w = *reinterpret_cast<const float2*>(par + 3 * kChunk + (2 * ib + j) * 8 + c2);
        float(&u)[4] = U[2 * ib + j];
        u[0] *= w.x; u[1] *= w.y; u[2] *= w.x; u[3] *= w.y;
      }
      uint32_t hi[4], lo[4];
      split_a(U[2 * ib], U[2 * ib + 1], hi, lo);
      const uint32_t ka = st + ((ib * 16 + at.row_t) * Sh::kRow + at.col_t) * 2;
#pragma unroll
      for (int np = 0; np < K / 16; np += 2) {
        uint32_t b[4], d[4];
        ldmatrix_x4_trans(b, ka + np * 32);
        ldmatrix_x4_trans(d, ka + np * 32 + 32);
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
    store_out(O, reinterpret_cast<__nv_bfloat16*>(stage + 2 * Sh::kK) + warp * 16, vrow,
              p.out + row0 * p.out_stride + static_cast<int64_t>(h) * p.V + p0 + warp * 16, p.out_stride,
              min(kChunk, n_tok - c * kChunk), pw - warp * 16, lane);
  }
  if (live && work) S.store(gS, p0 + warp * 16, p0 + pw, p.V, p.K, lane);
}

}  // namespace mv

// Bytes of scratch for a step, or -1 when the kernels do not take the sizes.
extern "C" int64_t mv_delta_chunk_workspace_bytes(int64_t tokens, int num_seqs, int heads, int dim, int vdim) {
  using namespace mv;
  if (tokens < 0 || num_seqs < 0 || heads <= 0 || !chunk_takes(dim, vdim)) return -1;
  return chunk_bound(tokens, num_seqs) * heads * kDcBytes;
}

extern "C" int mv_delta_chunk_scan(void* out, int64_t out_stride, const void* qkv, int64_t stride, const void* beta,
                                   const void* a, int64_t ba_stride, const void* A_log, const void* dt_bias,
                                   const int32_t* cu, int num_seqs, int64_t tokens, const int32_t* slots,
                                   const int32_t* start, float* state, int num_slots, int heads, int kv_heads, int dim,
                                   int vdim, float q_scale, void* workspace, int64_t workspace_bytes, void* stream) {
  using namespace mv;
  if (num_seqs < 0 || tokens < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || heads > 65535 || !chunk_takes(dim, vdim))
    return fail(MV_ERR_SHAPE, "delta_chunk_scan: heads %d over %d, dim %d, vdim %d", heads, kv_heads, dim, vdim);
  if (num_seqs == 0 || tokens == 0) return MV_OK;
  if (!out || !qkv || !beta || !a || !A_log || !dt_bias || !cu || !slots || !start || !state) return fail(MV_ERR_NULL, "delta_chunk_scan: null pointer");
  if (!vec8_ok(out, out_stride, 2) || !vec8_ok(qkv, stride, 2)) return fail(MV_ERR_ALIGN, "delta_chunk_scan: rows must start on 16-byte boundaries");
  const int64_t chunks = chunk_bound(tokens, num_seqs);
  if (!workspace || !aligned16(workspace) || workspace_bytes < chunks * heads * kDcBytes) return fail(MV_ERR_WORKSPACE, "delta_chunk_scan: workspace");
  auto c = [](const void* x) { return static_cast<const __nv_bfloat16*>(x); };
  const DeltaChunkParams p{static_cast<__nv_bfloat16*>(out), out_stride, c(qkv), stride, c(beta), c(a), ba_stride, c(A_log), c(dt_bias),
                           cu, slots, start, num_seqs, state, num_slots, heads, kv_heads, dim, vdim, q_scale,
                           static_cast<unsigned char*>(workspace)};
  auto st = static_cast<cudaStream_t>(stream);
  return chunk_dispatch(dim, [&](auto kk) {
    constexpr int K = decltype(kk)::value;
    constexpr int prep = DeltaPrepShape<K>::kBytes;
    cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel<K>, cudaFuncAttributeMaxDynamicSharedMemorySize, prep);
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "delta_chunk_scan: %s", cudaGetErrorString(e));
    delta_prepare_kernel<K><<<dim3(static_cast<unsigned>(chunks), kv_heads), kDpThreads, prep, st>>>(p);
    int rc = check_launch("delta_prepare");
    if (rc) return rc;
    const int pb = chunk_columns(static_cast<int64_t>(num_seqs) * heads, vdim), smem = 2 * DeltaChunkShape<K>::stage(pb);
    e = cudaFuncSetAttribute(delta_chunk_kernel<K>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "delta_chunk_scan: %s", cudaGetErrorString(e));
    delta_chunk_kernel<K><<<dim3(num_seqs, heads, (vdim + pb - 1) / pb), kChunkThreads, smem, st>>>(p, pb);
    return check_launch("delta_chunk");
  });
}
