// Chunked form of the selective recurrence for prompts, bf16 operands on tensor cores, fp32 state.
//
// One CTA walks the tokens of a (sequence, head, block of value columns) in chunks of 64, with the state S (N x P) as
// fp32 accumulators in registers.  With c_t the running sum of the log decays inside the chunk:
//   Y = exp(c_t) (C S_prev) + (M X) + D X,   M[t, j] = exp(c_t - c_j) dt_j (C_t . B_j) for j <= t
//   S = exp(c_last) S_prev + B^T (W X),       W_t = exp(c_last - c_t) dt_t
// C, B and X are the bf16 outputs of the convolution and enter the products as they are.  What the recurrence forms
// itself (M, W X, S) is fp32 and enters a product as two bf16 terms, the value and its rounding residue, so that the
// products carry 16 bits of it and nothing of the state is rounded to bf16.
// Two CTAs per SM: one computes while the other waits for its loads.
//
// Bytes per token and head: (2 * P + 2 * N / heads_per_group) * 2 + 2; the state is touched once per sequence.
#include <algorithm>
#include "mma.cuh"
#include "vec.cuh"

namespace mv {

constexpr int kCsThreads = 256, kCsQ = 64;

template <int N, int PB> struct CsShape {
  static constexpr int kXs = PB + 8, kBs = (N > PB ? N : PB) + 8, kMs = kCsQ + 8;  // row strides, elements (Y passes through C)
  static constexpr int kX = kCsQ * kXs, kB = kCsQ * kBs, kS = N * kXs;
  static constexpr int kM2 = 2 * kCsQ * kMs;                                      // M (two terms), later the residue of W X
  static_assert(kM2 >= kX, "the residue of W X lies over M");
  static constexpr int kElems = kX + 2 * kB + kM2 + 2 * kS;
  static constexpr int kBytes = kElems * 2;
};

struct CsParams {
  __nv_bfloat16* y; int64_t y_stride;
  const __nv_bfloat16* xbc; int64_t xbc_stride;
  const __nv_bfloat16* dt; int64_t dt_stride;
  const __nv_bfloat16 *dt_bias, *A_log, *D;
  const int32_t *cu, *slots, *start;
  float* state; int num_slots, heads, P, groups;
};

using Mma = Mma16816<__nv_bfloat16>;
template <int N, int PB>
__global__ void __launch_bounds__(kCsThreads, 2) ssm_chunk_kernel(const CsParams p) {
  using Sh = CsShape<N, PB>;
  constexpr int MT = N / 16;                          // 16-row tiles of the state
  constexpr int WPM = MT >= 8 ? 1 : 8 / MT;           // warps sharing a row tile (they split the columns)
  constexpr int MPW = MT >= 8 ? MT / 8 : 1;           // row tiles per warp
  constexpr int SN = PB / 8 / WPM;                    // 8-column tiles of the state per warp and row tile
  constexpr int YN = PB / 16;                         // 8-column tiles of Y per warp (four row tiles x two halves)
  static_assert(SN >= 1, "more warps than column tiles");
  extern __shared__ __align__(128) __nv_bfloat16 sm[];
  __nv_bfloat16 *sX = sm, *sB = sX + Sh::kX, *sC = sB + Sh::kB, *sM = sC + Sh::kB, *sS = sM + Sh::kM2;
  __shared__ __align__(8) float s_dts[2][kCsQ], s_cs[2][kCsQ];     // step sizes and running log2 decays of this chunk and the next
  const int s = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * PB, pw = min(PB, p.P - p0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = h / (p.heads / p.groups), inner = p.heads * p.P;
  const int slot = p.slots[s], st0 = p.start[s];
  const bool live = slot >= 0 && slot < p.num_slots && st0 >= 0;
  const int first = p.cu[s], n_tok = p.cu[s + 1] - first;
  if (n_tok <= 0) return;
  float* gS = p.state + (static_cast<int64_t>(live ? slot : 0) * p.heads + h) * N * p.P + p0;

  const int r8 = lane >> 2, c2 = (lane & 3) * 2;
  const int sm0 = MT >= 8 ? warp * MPW : warp / WPM;  // first state row tile of this warp
  const int sn0 = MT >= 8 ? 0 : (warp % WPM) * SN;    // its first column tile
  float S[MPW][SN][4];
#pragma unroll
  for (int a = 0; a < MPW; ++a)
#pragma unroll
    for (int b = 0; b < SN; ++b)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = (sm0 + a) * 16 + r8 + (e >> 1) * 8, q = (sn0 + b) * 8 + c2 + (e & 1);
        S[a][b][e] = live && st0 > 0 && q < pw ? gS[static_cast<int64_t>(n) * p.P + q] : 0.f;
      }
  auto store_S = [&] {      // both bf16 terms of S to shared memory, for the product with C
#pragma unroll
    for (int a = 0; a < MPW; ++a)
#pragma unroll
      for (int b = 0; b < SN; ++b)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t hi, lo;
          split2(S[a][b][half * 2], S[a][b][half * 2 + 1], hi, lo);
          const int at = ((sm0 + a) * 16 + r8 + half * 8) * Sh::kXs + (sn0 + b) * 8 + c2;
          *reinterpret_cast<uint32_t*>(sS + at) = hi;
          *reinterpret_cast<uint32_t*>(sS + Sh::kS + at) = lo;
        }
  };
  store_S();
  const float a2 = -expf(__bfloat162float(p.A_log[h])) * 1.4426950408889634f;
  const float db = __bfloat162float(p.dt_bias[h]), dd = __bfloat162float(p.D[h]);
  const uint32_t x_s = smem_u32(sX), b_s = smem_u32(sB), c_s = smem_u32(sC), m_s = smem_u32(sM), st_s = smem_u32(sS);
  const int l7 = lane & 7, l8 = (lane >> 3) & 1, l16 = lane >> 4;
  const int ym = warp >> 1, yn = warp & 1;            // this warp's 16 rows and half of the columns of G and Y

  // this thread's pieces of a chunk, as pointers that move from chunk to chunk
  constexpr int XC = PB / 8, XR = kCsQ * XC / kCsThreads, BC = N / 8, BR = kCsQ * BC / kCsThreads;
  static_assert(XR >= 1 && BR >= 1, "a chunk is at least one piece per thread");
  const int xt = tid / XC, xc = (tid % XC) * 8, bt0 = tid / BC, bc = (tid % BC) * 8, c_off = p.groups * N;
  const __nv_bfloat16* x_src = p.xbc + static_cast<int64_t>(first + xt) * p.xbc_stride + h * p.P + p0 + xc;
  const __nv_bfloat16* b_src = p.xbc + static_cast<int64_t>(first + bt0) * p.xbc_stride + inner + g * N + bc;
  __nv_bfloat16* y_dst = p.y + static_cast<int64_t>(first + xt) * p.y_stride + h * p.P + p0 + xc;
  const __nv_bfloat16* ahead = p.xbc + static_cast<int64_t>(first + kCsQ + (tid >> 2)) * p.xbc_stride +
      ((tid & 3) == 0 ? h * p.P + p0 : inner + ((tid & 3) == 2 ? p.groups + g : g) * N + ((tid & 3) == 3 ? N / 2 : 0));
  // dt: warp 0 reads a chunk's values while the chunk before it is worked on, two tokens per lane
  __nv_bfloat16 raw[2] = {__float2bfloat16_rn(0.f), __float2bfloat16_rn(0.f)};     // converted when used: nobody waits for the load
  auto fetch_dt = [&](int t0) {
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (t0 + lane * 2 + i < n_tok) raw[i] = p.dt[(static_cast<int64_t>(first) + t0 + lane * 2 + i) * p.dt_stride + h];
  };
  auto make_dt = [&](int t0) {
    float d[2], c[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      d[i] = t0 + lane * 2 + i < n_tok ? softplus_f(__bfloat162float(raw[i]) + db) : 0.f;
      c[i] = a2 * d[i];
    }
    float run = c[0] + c[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += v;
    }
    const int at = (t0 / kCsQ) & 1;
    s_dts[at][lane * 2] = d[0];
    s_dts[at][lane * 2 + 1] = d[1];
    s_cs[at][lane * 2] = run - c[1];
    s_cs[at][lane * 2 + 1] = run;
  };
  if (warp == 0) {
    fetch_dt(0);
    make_dt(0);
  }
  for (int t0 = 0; t0 < n_tok; t0 += kCsQ) {
    const int nt = min(kCsQ, n_tok - t0);
#pragma unroll
    for (int i = 0; i < XR; ++i) {
      const int t = xt + i * (kCsThreads / XC);
      const bool ok = t < nt && xc < pw;
      cp_async16(x_s + (t * Sh::kXs + xc) * 2, ok ? x_src + i * (kCsThreads / XC) * p.xbc_stride : p.xbc, ok ? 16 : 0);
    }
#pragma unroll
    for (int i = 0; i < BR; ++i) {
      const int t = bt0 + i * (kCsThreads / BC);
      const bool ok = t < nt;
      const __nv_bfloat16* src = ok ? b_src + i * (kCsThreads / BC) * p.xbc_stride : p.xbc;
      cp_async16(b_s + (t * Sh::kBs + bc) * 2, src, ok ? 16 : 0);
      cp_async16(c_s + (t * Sh::kBs + bc) * 2, ok ? src + c_off : src, ok ? 16 : 0);
    }
    cp_async_commit();
    x_src += kCsQ * p.xbc_stride;
    b_src += kCsQ * p.xbc_stride;
    {  // the next chunk's lines on their way to L2
      const int t = tid >> 2, part = tid & 3;
      if (t0 + kCsQ + t < n_tok) {
        asm volatile("prefetch.global.L2 [%0];" ::"l"(ahead));
        if (part == 2 && N > 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(ahead + N / 2));
      }
      ahead += kCsQ * p.xbc_stride;
    }
    const int cur = (t0 / kCsQ) & 1;
    const float *s_dt = s_dts[cur], *s_c = s_cs[cur];
    if (warp == 0) fetch_dt(t0 + kCsQ);
    cp_async_wait<0>();
    __syncthreads();

    float acc[YN][4];
    const float ct0 = s_c[ym * 16 + r8], ct1 = s_c[ym * 16 + r8 + 8];
    {  // G = C B^T for this warp's 16 x 32 block, then M in two terms
      const bool need = yn * 32 <= ym * 16 + 15;
      float G[4][4] = {};
      if (need) {
        const uint32_t ca = c_s + ((ym * 16 + l7 + l8 * 8) * Sh::kBs + l16 * 8) * 2;
        const uint32_t ba = b_s + ((yn * 32 + l7 + l16 * 8) * Sh::kBs + l8 * 8) * 2;
#pragma unroll
        for (int k = 0; k < N; k += 16) {
          uint32_t a[4], b[4];
          ldmatrix_x4(a, ca + k * 2);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            ldmatrix_x4(b, ba + (j * 16 * Sh::kBs + k) * 2);
            Mma::run(G[2 * j], a, b[0], b[1]);
            Mma::run(G[2 * j + 1], a, b[2], b[3]);
          }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int col = yn * 32 + j * 8 + c2;
          const float2 cj = *reinterpret_cast<const float2*>(s_c + col), dj = *reinterpret_cast<const float2*>(s_dt + col);
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int row = ym * 16 + r8 + half * 8;
            const float ct = half ? ct1 : ct0;
            const float m0 = col <= row ? G[j][half * 2] * fast_exp2(ct - cj.x) * dj.x : 0.f;
            const float m1 = col + 1 <= row ? G[j][half * 2 + 1] * fast_exp2(ct - cj.y) * dj.y : 0.f;
            uint32_t hi, lo;
            split2(m0, m1, hi, lo);
            *reinterpret_cast<uint32_t*>(sM + row * Sh::kMs + col) = hi;
            *reinterpret_cast<uint32_t*>(sM + kCsQ * Sh::kMs + row * Sh::kMs + col) = lo;
          }
        }
      }
    }
    {  // C S_prev, scaled by the decay since the chunk's start
#pragma unroll
      for (int i = 0; i < YN; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
      const uint32_t ca = c_s + ((ym * 16 + l7 + l8 * 8) * Sh::kBs + l16 * 8) * 2;
      const uint32_t sa = st_s + ((l7 + l8 * 8) * Sh::kXs + yn * (PB / 2) + l16 * 8) * 2;
#pragma unroll
      for (int k = 0; k < N; k += 16) {
        uint32_t a[4], b[4];
        ldmatrix_x4(a, ca + k * 2);
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int i = 0; i < YN; i += 2) {
            ldmatrix_x4_trans(b, sa + (term * Sh::kS + k * Sh::kXs + i * 8) * 2);
            Mma::run(acc[i], a, b[0], b[1]);
            Mma::run(acc[i + 1], a, b[2], b[3]);
          }
      }
      const float e0 = fast_exp2(ct0), e1 = fast_exp2(ct1);
#pragma unroll
      for (int i = 0; i < YN; ++i) {
        acc[i][0] *= e0; acc[i][1] *= e0; acc[i][2] *= e1; acc[i][3] *= e1;
      }
    }
    __syncthreads();                       // M is complete; C and S have been read
    {  // + M X + D X
      const uint32_t ma = m_s + ((ym * 16 + l7 + l8 * 8) * Sh::kMs + l16 * 8) * 2;
      const uint32_t xa = x_s + ((l7 + l8 * 8) * Sh::kXs + yn * (PB / 2) + l16 * 8) * 2;
      for (int k = 0; k <= ym * 16; k += 16) {
        uint32_t hi[4], lo[4], b[4];
        ldmatrix_x4(hi, ma + k * 2);
        ldmatrix_x4(lo, ma + (kCsQ * Sh::kMs + k) * 2);
#pragma unroll
        for (int i = 0; i < YN; i += 2) {
          ldmatrix_x4_trans(b, xa + (k * Sh::kXs + i * 8) * 2);
          Mma::run(acc[i], hi, b[0], b[1]);
          Mma::run(acc[i + 1], hi, b[2], b[3]);
          Mma::run(acc[i], lo, b[0], b[1]);
          Mma::run(acc[i + 1], lo, b[2], b[3]);
        }
      }
      // Y goes to global memory through the buffer of C, whole rows at a time
#pragma unroll
      for (int i = 0; i < YN; ++i)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int row = ym * 16 + r8 + half * 8, col = yn * (PB / 2) + i * 8 + c2;
          const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sX + row * Sh::kXs + col));
          const __nv_bfloat162 v = __floats2bfloat162_rn(fmaf(dd, x.x, acc[i][half * 2]), fmaf(dd, x.y, acc[i][half * 2 + 1]));
          *reinterpret_cast<__nv_bfloat162*>(sC + row * Sh::kBs + col) = v;
        }
    }
    if (warp == 0) make_dt(t0 + kCsQ);     // its rows have the fewest products
    __syncthreads();                       // M has been read, Y is complete
    const float cl = s_c[kCsQ - 1];
    for (int i = tid; i < kCsQ * (PB / 8); i += kCsThreads) {    // W X in two terms: the value in place, the residue over M
      const int t = i / (PB / 8), c = (i % (PB / 8)) * 8;
      const float w = fast_exp2(cl - s_c[t]) * s_dt[t];
      float v[8], lo[8];
      Vec<__nv_bfloat16, 8>::load(sX + t * Sh::kXs + c, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        v[e] *= w;
        lo[e] = v[e] - __bfloat162float(__float2bfloat16_rn(v[e]));
      }
      Vec<__nv_bfloat16, 8>::store(sX + t * Sh::kXs + c, v);
      Vec<__nv_bfloat16, 8>::store(sM + t * Sh::kXs + c, lo);
    }
#pragma unroll
    for (int i = 0; i < XR; ++i) {
      const int t = xt + i * (kCsThreads / XC);
      if (t < nt && xc < pw)
        *reinterpret_cast<uint4*>(y_dst + i * (kCsThreads / XC) * p.y_stride) = *reinterpret_cast<const uint4*>(sC + t * Sh::kBs + xc);
    }
    y_dst += kCsQ * p.y_stride;
    __syncthreads();
    {  // S = exp(c_last) S + (W B)^T X
      const float e = fast_exp2(cl);
#pragma unroll
      for (int a = 0; a < MPW; ++a)
#pragma unroll
        for (int b = 0; b < SN; ++b)
#pragma unroll
          for (int q = 0; q < 4; ++q) S[a][b][q] *= e;
      const uint32_t xo = ((l7 + l8 * 8) * Sh::kXs + sn0 * 8 + l16 * 8) * 2;
#pragma unroll
      for (int k = 0; k < kCsQ; k += 16) {
        uint32_t bt[MPW][4];
#pragma unroll
        for (int a = 0; a < MPW; ++a)
          ldmatrix_x4_trans(bt[a], b_s + ((k + l7 + l16 * 8) * Sh::kBs + (sm0 + a) * 16 + l8 * 8) * 2);
#pragma unroll
        for (int i = 0; i < SN; i += 2) {
          uint32_t hi[4], lo[4];
          ldmatrix_x4_trans(hi, x_s + xo + (k * Sh::kXs + i * 8) * 2);
          ldmatrix_x4_trans(lo, m_s + xo + (k * Sh::kXs + i * 8) * 2);
#pragma unroll
          for (int a = 0; a < MPW; ++a) {
            Mma::run(S[a][i], bt[a], hi[0], hi[1]);
            if (i + 1 < SN) Mma::run(S[a][i + 1 < SN ? i + 1 : i], bt[a], hi[2], hi[3]);
            Mma::run(S[a][i], bt[a], lo[0], lo[1]);
            if (i + 1 < SN) Mma::run(S[a][i + 1 < SN ? i + 1 : i], bt[a], lo[2], lo[3]);
          }
        }
      }
      store_S();
    }
    __syncthreads();                       // every buffer is free for the next chunk
  }
  if (!live) return;
#pragma unroll
  for (int a = 0; a < MPW; ++a)
#pragma unroll
    for (int b = 0; b < SN; ++b)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = (sm0 + a) * 16 + r8 + (e >> 1) * 8, q = (sn0 + b) * 8 + c2 + (e & 1);
        if (q < pw) gS[static_cast<int64_t>(n) * p.P + q] = S[a][b][e];
      }
}

template <int N, int PB> static int launch_chunk(const CsParams& p, int num_seqs, cudaStream_t st) {
  const int smem = CsShape<N, PB>::kBytes;
  const cudaError_t e = cudaFuncSetAttribute(ssm_chunk_kernel<N, PB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return fail(MV_ERR_CUDA, "ssm_chunk_scan: %s", cudaGetErrorString(e));
  ssm_chunk_kernel<N, PB><<<dim3(num_seqs, p.heads, (p.P + PB - 1) / PB), kCsThreads, smem, st>>>(p);
  return check_launch("ssm_chunk_scan");
}

}  // namespace mv

// Does the chunked kernel take this state size and value size?
extern "C" int mv_ssm_chunk_takes(int vdim, int state_dim) {
  return (state_dim == 32 || state_dim == 64 || state_dim == 128) && vdim > 0 && vdim % 8 == 0;
}

extern "C" int mv_ssm_chunk_scan(void* y, int64_t y_stride, const void* xbc, int64_t xbc_stride, const void* dt,
                                 int64_t dt_stride, const void* dt_bias, const void* A_log, const void* D,
                                 const int32_t* cu, int num_seqs, const int32_t* slots, const int32_t* start,
                                 float* state, int num_slots, int heads, int vdim, int state_dim, int groups,
                                 void* stream) {
  using namespace mv;
  if (num_seqs < 0 || heads <= 0 || groups <= 0 || heads % groups || !mv_ssm_chunk_takes(vdim, state_dim))
    return fail(MV_ERR_SHAPE, "ssm_chunk_scan: heads %d groups %d vdim %d state %d", heads, groups, vdim, state_dim);
  if (num_seqs == 0) return MV_OK;
  if (!y || !xbc || !dt || !dt_bias || !A_log || !D || !cu || !slots || !start || !state)
    return fail(MV_ERR_NULL, "ssm_chunk_scan: null pointer");
  if (!vec8_ok(y, y_stride, 2) || !vec8_ok(xbc, xbc_stride, 2)) return fail(MV_ERR_ALIGN, "ssm_chunk_scan: rows must start on 16-byte boundaries");
  const CsParams p{static_cast<__nv_bfloat16*>(y), y_stride, static_cast<const __nv_bfloat16*>(xbc), xbc_stride,
                   static_cast<const __nv_bfloat16*>(dt), dt_stride, static_cast<const __nv_bfloat16*>(dt_bias),
                   static_cast<const __nv_bfloat16*>(A_log), static_cast<const __nv_bfloat16*>(D), cu, slots, start, state,
                   num_slots, heads, vdim, groups};
  auto st = static_cast<cudaStream_t>(stream);
  // few (sequence, head) pairs: narrower column blocks, so that more SMs have work
  const bool narrow = vdim <= 32 || static_cast<int64_t>(num_seqs) * heads * ((vdim + 63) / 64) < 2 * kNumSMs;
  auto go = [&](auto n) {
    constexpr int N = decltype(n)::value;
    return narrow ? launch_chunk<N, 32>(p, num_seqs, st) : launch_chunk<N, 64>(p, num_seqs, st);
  };
  if (state_dim == 32) return go(std::integral_constant<int, 32>{});
  if (state_dim == 64) return go(std::integral_constant<int, 64>{});
  return go(std::integral_constant<int, 128>{});
}
