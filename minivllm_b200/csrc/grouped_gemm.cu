// Grouped matrix product of a mixture of experts on the Blackwell tensor cores: rows [offsets[e], offsets[e + 1])
// of x (sorted by expert) times w[e]^T, bf16 in and out, fp32 accumulation in tensor memory.
//
// The weights are the M side (128 output features = 128 TMEM lanes), the tokens the N side, so that a decode step
// with a handful of tokens per expert wastes no tensor-core rows and streams each weight once, and a prefill step
// uses the same kernel with 128-token tiles.  A unit of work is two 128-feature tiles times one token tile: the gate
// and up rows of the same features (kGated: the epilogue applies the gate, glu_act), or 256 consecutive features.
// Persistent CTAs walk the units of all experts in order; unit ranges come from the device-side offsets.
//   warps 0-3  epilogue: accumulators -> registers -> global (a store instruction covers 32 consecutive features)
//   warp 4     TMA producer: two weight tiles and a token tile per 64-deep slab, ring of kStages
//   warp 5     MMA issuer
// Two accumulator sets: the epilogue of one unit runs beside the products of the next.
//
// Prefill: tensor-bound, FLOPs = 2 * rows * in * out (* 2 gated).  Decode: HBM-bound on the weights of the experts
// that have tokens.
#include <algorithm>
#include "tcgen05.cuh"
#include "tmap.cuh"
#include "vec.cuh"

namespace mv {

constexpr int kGmThreads = 192;
constexpr int kGmTile = 128 * 128;       // bytes of a 128-row, 64-column bf16 tile
constexpr int kGmMaxExperts = 1024;
template <int NT> struct GmShape {
  static constexpr int kStages = NT == 128 ? 4 : NT == 64 ? 5 : 6;
  static constexpr int kStageBytes = 2 * kGmTile + NT * 128;
  static constexpr int kCols = NT == 16 ? 128 : 4 * NT;    // two sets of two accumulators
  static constexpr int kSmem = kStages * kStageBytes + 1024;
};

struct GmParams {
  __nv_bfloat16* out;
  const int32_t* offsets;
  int experts, in_dim, out_dim, out_tiles;
  int act;
  float limit;
  int* error_word;
};

enum { GB_FULL = 0, GB_EMPTY = 8, GB_AFULL = 16, GB_AEMPTY = 18, GB_DRAIN = 20, GB_COUNT = 21 };

struct GmUnit { int e, o0, row0, rows; };
// Unit u: expert by binary search in the prefix sums of units; within an expert the token tile runs fastest, so that
// CTAs working side by side read the same weights.
template <int NT>
__device__ __forceinline__ GmUnit gm_unit(const int* start, const GmParams& p, int u, int step) {
  int lo = 0, hi = p.experts - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (start[mid] <= u) lo = mid; else hi = mid - 1;
  }
  const int first = p.offsets[lo], n = p.offsets[lo + 1] - first, tt = (n + NT - 1) / NT;
  const int v = u - start[lo], ot = v / tt, t = v - ot * tt;
  return GmUnit{lo, ot * step, first + t * NT, min(NT, n - t * NT)};
}

template <int NT, bool kGated>
__global__ void __launch_bounds__(kGmThreads, 1)
grouped_gemm_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x,
                    const GmParams p) {
  using Sh = GmShape<NT>;
  constexpr int kStep = kGated ? 128 : 256;      // output features per unit
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t bars[GB_COUNT];
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort, s_sticky;
  __shared__ int s_start[kGmMaxExperts + 1];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t smem = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t bar0 = smem_u32(bars);
  auto bar = [&](int i) { return bar0 + 8u * i; };
  volatile int* abort_flag = &s_abort;

  if (tid == 0) {
    s_abort = 0;
    s_sticky = *reinterpret_cast<volatile int*>(p.error_word);
    for (int i = 0; i < Sh::kStages; ++i) {
      tc::mbar_init(bar(GB_FULL + i), 1);
      tc::mbar_init(bar(GB_EMPTY + i), 1);
    }
    for (int i = 0; i < 2; ++i) {
      tc::mbar_init(bar(GB_AFULL + i), 1);
      tc::mbar_init(bar(GB_AEMPTY + i), 128);
    }
    tc::mbar_init(bar(GB_DRAIN), 1);
    tc::mbar_fence_init();
  }
  if (warp == 0) {       // prefix sums of units over the experts
    int carry = 0;
    for (int b = 0; b < p.experts; b += 32) {
      const int e = b + lane;
      const int n = e < p.experts ? (p.offsets[e + 1] - p.offsets[e] + NT - 1) / NT * p.out_tiles : 0;
      int incl = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += v;
      }
      if (e < p.experts) s_start[e] = carry + incl - n;
      carry += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (lane == 0) s_start[p.experts] = carry;
  }
  if (warp == 5) {
    tc::tmem_alloc(smem_u32(&s_tmem), Sh::kCols);
    tc::tmem_relinquish();
  }
  tc::fence_before_sync();
  __syncthreads();
  tc::fence_after_sync();
  const uint32_t tmem = s_tmem;
  const int units = s_sticky == 0 ? s_start[p.experts] : 0;    // an earlier wait that ran out: do nothing
  const int slabs = (p.in_dim + 63) / 64;

  if (warp == 4) {
    if (lane == 0) {
      tc::tma_prefetch_desc(&tmap_w);
      tc::tma_prefetch_desc(&tmap_x);
      uint32_t it = 0;
      bool ok = true;
      for (int u = blockIdx.x; u < units && ok; u += gridDim.x) {
        const GmUnit un = gm_unit<NT>(s_start, p, u, kStep);
        const int wrow = un.e * (kGated ? 2 : 1) * p.out_dim + un.o0;
        const bool two = kGated || un.o0 + 128 < p.out_dim;
        const int second = kGated ? wrow + p.out_dim : wrow + 128;
        for (int k = 0; k < slabs; ++k, ++it) {
          const int s = it % Sh::kStages;
          if (it >= Sh::kStages && !tc::mbar_wait(bar(GB_EMPTY + s), (it / Sh::kStages - 1) & 1, abort_flag, p.error_word, 0x40)) {
            ok = false;
            break;
          }
          const uint32_t st = smem + s * Sh::kStageBytes;
          tc::mbar_expect_tx(bar(GB_FULL + s), (two ? 2 : 1) * kGmTile + NT * 128);
          tc::tma_load_3d(st, &tmap_w, k * 64, wrow, 0, bar(GB_FULL + s));
          if (two) tc::tma_load_3d(st + kGmTile, &tmap_w, k * 64, second, 0, bar(GB_FULL + s));
          tc::tma_load_3d(st + 2 * kGmTile, &tmap_x, k * 64, un.row0, 0, bar(GB_FULL + s));
        }
      }
      if (!ok)             // copies in flight must land before the CTA's shared memory goes away
        for (uint32_t i = it >= Sh::kStages ? it - Sh::kStages : 0; i < it; ++i)
          tc::mbar_wait_timed(bar(GB_FULL + i % Sh::kStages), (i / Sh::kStages) & 1);
    }
  } else if (warp == 5) {
    const uint32_t idesc = tc::instr_desc_f16(1, 1, false, 128, NT);
    uint32_t it = 0, n = 0;
    bool ok = true;
    for (int u = blockIdx.x; u < units && ok; u += gridDim.x, ++n) {
      const GmUnit un = gm_unit<NT>(s_start, p, u, kStep);
      const bool two = kGated || un.o0 + 128 < p.out_dim;
      const int b = n & 1;
      if (n >= 2 && !tc::mbar_wait(bar(GB_AEMPTY + b), (n / 2 - 1) & 1, abort_flag, p.error_word, 0x41)) { ok = false; break; }
      tc::fence_after_sync();
      const uint32_t d = tmem + b * 2 * NT;
      for (int k = 0; k < slabs; ++k, ++it) {
        const int s = it % Sh::kStages;
        if (!tc::mbar_wait(bar(GB_FULL + s), (it / Sh::kStages) & 1, abort_flag, p.error_word, 0x42)) { ok = false; break; }
        tc::fence_after_sync();
        const uint32_t st = smem + s * Sh::kStageBytes;
        const uint64_t da = tc::desc64(tc::desc_lo(st, 16), tc::kDescHiSw128Sbo1024);
        const uint64_t db = tc::desc64(tc::desc_lo(st + 2 * kGmTile, 16), tc::kDescHiSw128Sbo1024);
        __syncwarp();
        tc::mma_ss_k64(d, da, db, idesc, k > 0);
        if (two) tc::mma_ss_k64(d + NT, da + (kGmTile >> 4), db, idesc, k > 0);
        tc::commit_elected(bar(GB_EMPTY + s), bar(GB_AFULL + b), k == slabs - 1);
      }
    }
    if (!ok) {
      __syncwarp();
      tc::commit_elected(bar(GB_DRAIN), bar(GB_DRAIN), false);
      tc::mbar_wait_timed(bar(GB_DRAIN), 0);
    }
  } else {
    uint32_t n = 0;
    for (int u = blockIdx.x; u < units; u += gridDim.x, ++n) {
      const GmUnit un = gm_unit<NT>(s_start, p, u, kStep);
      const int b = n & 1;
      if (!tc::mbar_wait(bar(GB_AFULL + b), (n / 2) & 1, abort_flag, p.error_word, 0x43)) break;
      tc::fence_after_sync();
      const uint32_t d = tmem + b * 2 * NT + (static_cast<uint32_t>(warp * 32) << 16);
      const int o = un.o0 + warp * 32 + lane;
      constexpr int kChunk = NT < 32 ? NT : 32;
#pragma unroll 1
      for (int j0 = 0; j0 < NT; j0 += kChunk) {
        if (j0 >= un.rows) break;
        __nv_bfloat16* dst = p.out + static_cast<int64_t>(un.row0 + j0) * p.out_dim + o;
        const int lim = un.rows - j0;
        uint32_t a[32], c[32];
        tc::tmem_ld32(d + j0, a);
        if (kGated || un.o0 + 128 < p.out_dim) tc::tmem_ld32(d + NT + j0, c);
        tc::wait_ld();
        if (kGated) {
          if (o < p.out_dim) {
            auto apply = [&](auto act) {
#pragma unroll
              for (int j = 0; j < kChunk; ++j)
                if (j < lim)
                  dst[static_cast<int64_t>(j) * p.out_dim] = __float2bfloat16_rn(
                      glu_act<__nv_bfloat16>(decltype(act)::value, __uint_as_float(a[j]), __uint_as_float(c[j]), p.limit));
            };
            switch (p.act) {
              case MV_ACT_SILU: apply(std::integral_constant<int, MV_ACT_SILU>{}); break;
              case MV_ACT_SIGMOID: apply(std::integral_constant<int, MV_ACT_SIGMOID>{}); break;
              case MV_ACT_GELU_TANH: apply(std::integral_constant<int, MV_ACT_GELU_TANH>{}); break;
              case MV_ACT_RELU: apply(std::integral_constant<int, MV_ACT_RELU>{}); break;
              default: apply(std::integral_constant<int, MV_ACT_CLAMPED>{});
            }
          }
        } else {
          if (o < p.out_dim) {
#pragma unroll
            for (int j = 0; j < kChunk; ++j)
              if (j < lim) dst[static_cast<int64_t>(j) * p.out_dim] = __float2bfloat16_rn(__uint_as_float(a[j]));
          }
          if (o + 128 < p.out_dim) {
#pragma unroll
            for (int j = 0; j < kChunk; ++j)
              if (j < lim) dst[static_cast<int64_t>(j) * p.out_dim + 128] = __float2bfloat16_rn(__uint_as_float(c[j]));
          }
        }
      }
      tc::fence_before_sync();
      tc::mbar_arrive(bar(GB_AEMPTY + b));
    }
  }
  __syncwarp();
  tc::fence_before_sync();
  __syncthreads();
  if (warp == 5) {
    tc::fence_after_sync();
    tc::tmem_dealloc(tmem, Sh::kCols);
  }
}

template <int NT, bool kGated>
static int launch_grouped(const CUtensorMap& tw, const void* x, int64_t rows, GmParams p, cudaStream_t st) {
  CUtensorMap tx;
  int rc = make_tmap_bf16(&tx, x, p.in_dim, rows, 1, p.in_dim, rows * p.in_dim, NT, 1, "grouped_gemm");
  if (rc) return rc;
  const cudaError_t e = cudaFuncSetAttribute(grouped_gemm_kernel<NT, kGated>, cudaFuncAttributeMaxDynamicSharedMemorySize, GmShape<NT>::kSmem);
  if (e != cudaSuccess) return fail(MV_ERR_CUDA, "grouped_gemm: %s", cudaGetErrorString(e));
  const int64_t most = (rows / NT + std::min<int64_t>(p.experts, rows)) * p.out_tiles;
  const unsigned grid = static_cast<unsigned>(std::min<int64_t>(most, kNumSMs));
  grouped_gemm_kernel<NT, kGated><<<grid, kGmThreads, GmShape<NT>::kSmem, st>>>(tw, tx, p);
  return check_launch("grouped_gemm");
}

}  // namespace mv

extern "C" int mv_grouped_gemm(void* out, const void* x, const void* w, const int32_t* offsets, int experts,
                               int64_t rows, int in_dim, int out_dim, int act, float limit, int* error_word,
                               void* stream) {
  using namespace mv;
  if (act < MV_ACT_NONE || act > MV_ACT_RELU) return fail(MV_ERR_SHAPE, "grouped_gemm: activation %d", act);
  const bool gated = act != MV_ACT_NONE;
  if (rows < 0 || experts <= 0 || in_dim <= 0 || out_dim <= 0) return fail(MV_ERR_SHAPE, "grouped_gemm: %d x %d", out_dim, in_dim);
  if (in_dim % 8) return fail(MV_ERR_SHAPE, "grouped_gemm: in_dim %d is not a multiple of 8", in_dim);
  if (experts > kGmMaxExperts) return fail(MV_ERR_LIMIT, "grouped_gemm: %d experts (at most %d)", experts, kGmMaxExperts);
  if (rows > (1 << 28)) return fail(MV_ERR_LIMIT, "grouped_gemm: %lld rows", static_cast<long long>(rows));
  if (rows == 0) return MV_OK;
  if (!out || !x || !w || !offsets || !error_word) return fail(MV_ERR_NULL, "grouped_gemm: null pointer");
  if (!aligned16(x) || !aligned16(w)) return fail(MV_ERR_ALIGN, "grouped_gemm: operands must be 16-byte aligned");
  CUtensorMap tw;
  const int64_t wrows = static_cast<int64_t>(experts) * (gated ? 2 : 1) * out_dim;
  const int rc = make_tmap_bf16(&tw, w, in_dim, wrows, 1, in_dim, wrows * in_dim, 128, 1, "grouped_gemm");
  if (rc) return rc;
  GmParams p{static_cast<__nv_bfloat16*>(out), offsets, experts, in_dim, out_dim,
             gated ? (out_dim + 127) / 128 : (out_dim + 255) / 256, act, limit, error_word};
  auto st = static_cast<cudaStream_t>(stream);
  // token tile by the mean number of rows of an expert; an expert with more has several tiles
  const int64_t mean = (rows + experts - 1) / experts;
  auto go = [&](auto g) {
    constexpr bool G = decltype(g)::value;
    if (mean <= 12) return launch_grouped<16, G>(tw, x, rows, p, st);
    if (mean <= 28) return launch_grouped<32, G>(tw, x, rows, p, st);
    if (mean <= 64) return launch_grouped<64, G>(tw, x, rows, p, st);
    return launch_grouped<128, G>(tw, x, rows, p, st);
  };
  return gated ? go(std::integral_constant<bool, true>{}) : go(std::integral_constant<bool, false>{});
}
