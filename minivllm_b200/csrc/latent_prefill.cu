// Prefill attention on the Blackwell tensor cores, causal, packed batch, an optional sink per head, in three forms:
//   latent attention, with keys and values expanded per head (k = [W_uk c | shared rotated part], v = W_uv c);
//   kWin: grouped-query attention with a sliding window and a bias per distance and head; results may be turned back by
//   their positions in pairs of neighbouring columns (values that were turned when they were stored);
//   kDiff: differential attention in chunks of the sequence: a head has two maps over the same values.
//
// The two 128-row problems of a CTA are two consecutive query tiles of ONE head (latent attention: every head has keys of
// its own): they share each K/V tile.  The K operand is assembled by TMA from two tensors, 64-column boxes of the expanded
// unrotated part and one box of the rotated part that all heads share; a box that is wider than its tensor reads
// zeros, so any sizes that are multiples of eight up to 192 query/key and 128 value dimensions run here.
//   warps 0-3 / 4-7  softmax of the lower / upper query tile (thread = row = TMEM lane)
//   warp 8           TMA producer, warp 9 MMA issuer (S = Q K^T from shared memory, O += P V with P in TMEM)
// Sequence s has queries cu_q[s] .. and keys cu_k[s] .. of the packed tensors; its first query sits at position
// (keys - queries).  Same roles, tensor-memory layout and lazy rescaling as prefill_varlen.cu.
//
// kWin: K/V tiles outside both query tiles' windows are not visited.  The bias table of the head lies in shared memory by
// distance, from -256 on, with -inf where a distance is not visible, so that one lookup masks and biases a score; tiles
// whose distances all lie at or beyond the table's last entry add that entry instead.
//
// kDiff: the two problems are the two maps of one head on the same query tile; a K stage holds both maps' keys.  In the end each
// warpgroup takes half of the columns of both results: their difference, its norm over the head, and the output gate.
//
// Tensor-bound: FLOPs = 2 * heads * (dim + rot_dim + vdim) * (number of visible (query, key) pairs).
#include <algorithm>
#include "mma.cuh"
#include "query_tile.cuh"
#include "tcgen05.cuh"
#include "tmap.cuh"
#include "vec.cuh"

namespace mv {

constexpr int kLfThreads = 384, kLfTile = 128;
constexpr int kLfBox = kLfTile * 128;                 // one 64-column box of a 128-row tile
constexpr float kLfRescale = 8.f;                     // log2 units

constexpr int kLfBefore = 256, kLfAfter = 256;        // bias table: entries in front of distance 0 and past the last one

enum { LF_LATENT = 0, LF_WINDOW = 1, LF_DIFF = 2 };
template <int NQ, int NV, int FORM> struct LfShape {
  static constexpr bool kWin = FORM == LF_WINDOW, kDiff = FORM == LF_DIFF;
  static constexpr int kKStages = (kWin && NQ == 3) || (kDiff && NQ == 2) ? 1 : 2;
  static constexpr int kVStages = NQ == 3 && NV == 2 && !kWin ? 1 : 2;
  static constexpr int kQBytes = NQ * kLfBox, kKBytes = (kDiff ? 2 : 1) * kQBytes, kVBytes = NV * kLfBox;
  static constexpr int kSmem = 2 * kQBytes + kKStages * kKBytes + kVStages * kVBytes + 1024;
  static constexpr int kTable = (227 * 1024 - 512 - kSmem) / 4;       // floats left for the bias table
};

struct LfParams {
  __nv_bfloat16* out; int64_t out_stride; int vdim;
  const int32_t* cu_q; const int32_t* cu_k;
  int num_seqs, nd, dim, rot_dim;                     // nd: boxes of the unrotated part
  float scale_log2;
  const __nv_bfloat16* sink;
  int* error_word;
  int group;                                          // query heads per KV head
  int window, distances;                              // kWin; bias may be null
  const float* bias; int64_t bias_stride;
  const float2* turn; int64_t table_rows;             // kWin: (vdim / 2, table_rows) cos, sin; null: results stay as they are
  const int64_t* positions;                           // of the queries
  int chunk;                                          // kDiff
  const __nv_bfloat16* gate; int64_t gate_stride;
  float lambda, mult, eps;
};

enum { LB_Q = 0, LB_KFULL = 1, LB_KEMPTY = 3, LB_VFULL = 5, LB_VEMPTY = 7, LB_SFULL = 9, LB_PREADY = 11, LB_ODONE = 13,
       LB_DRAIN = 15, LB_COUNT = 16 };

// A pair of columns (fp32 bits) turned by the opposite of an angle, given as (cos, sin).
__device__ __forceinline__ void turn_back(uint32_t& a, uint32_t& b, float2 cs) {
  const float x = __uint_as_float(a), y = __uint_as_float(b);
  a = __float_as_uint(fmaf(x, cs.x, y * cs.y));
  b = __float_as_uint(fmaf(y, cs.x, -x * cs.y));
}

template <int NQ, int NV, int FORM>
__global__ void __launch_bounds__(kLfThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tm_qn, const __grid_constant__ CUtensorMap tm_qr,
                      const __grid_constant__ CUtensorMap tm_kn, const __grid_constant__ CUtensorMap tm_kr,
                      const __grid_constant__ CUtensorMap tm_v, const LfParams p) {
  using Sh = LfShape<NQ, NV, FORM>;
  constexpr bool kWin = Sh::kWin, kDiff = Sh::kDiff;
  constexpr int kRows = kDiff ? kLfTile : 2 * kLfTile, kSecond = kDiff ? 0 : kLfTile;      // queries of a CTA; where the second problem's begin
  constexpr int VS = Sh::kVStages, KS = Sh::kKStages;
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t bars[LB_COUNT];
  __shared__ uint32_t s_tmem;
  __shared__ int s_tile[2], s_scan[kLfThreads / 32], s_abort, s_sticky;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t q_smem = (smem_u32(smem_raw) + 1023u) & ~1023u;      // [tile 2][box][128][128B]
  const uint32_t k_smem = q_smem + 2 * Sh::kQBytes;                   // [stage KS][box]
  const uint32_t v_smem = k_smem + KS * Sh::kKBytes;                  // [stage VS][box]
  float* s_bias = reinterpret_cast<float*>(smem_raw + (v_smem + VS * Sh::kVBytes - smem_u32(smem_raw)));     // kWin
  const uint32_t bar0 = smem_u32(bars);
  auto bar = [&](int i) { return bar0 + 8u * i; };
  volatile int* abort_flag = &s_abort;

  if (tid == 0) {
    s_abort = 0;
    s_sticky = *reinterpret_cast<volatile int*>(p.error_word);
  }
  find_query_tile<kLfThreads>(p.cu_q, p.num_seqs, kRows, s_tile, s_scan);
  const int seq = s_tile[0];
  if (seq < 0 || s_sticky != 0) return;      // uniform: the grid is an upper bound; an earlier wait ran out
  const int head = blockIdx.y, kv_head = FORM == LF_LATENT ? head : head / p.group;
  const int q_start = p.cu_q[seq], q_len = p.cu_q[seq + 1] - q_start;
  const int k_start = p.cu_k[seq], k_len = p.cu_k[seq + 1] - k_start;
  const int q0 = s_tile[1] * kRows;
  const int first_pos = k_len - q_len + q0;
  // KV tiles up to the position of each query tile's last row
  const int n_a = (k_len - q_len + min(q0 + kLfTile, q_len) + kLfTile - 1) / kLfTile;
  const int n_b = kDiff ? n_a : q0 + kLfTile < q_len ? (k_len - q_len + min(q0 + 2 * kLfTile, q_len) + kLfTile - 1) / kLfTile : 0;
  const int n_kv = max(n_a, n_b);
  // kWin: first KV tile of each query tile; ring positions count from lo_a
  const int lo_a = kDiff ? first_pos / p.chunk * p.chunk / kLfTile : kWin ? min(max(first_pos - p.window + 1, 0) / kLfTile, n_a - 1) : 0;
  const int lo_b = kDiff ? lo_a : kWin && n_b > 0 ? max(first_pos + kLfTile - p.window + 1, 0) / kLfTile : 0;
  if (kWin)
    for (int i = tid; i < kLfBefore + p.distances + kLfAfter; i += kLfThreads) {
      const int d = i - kLfBefore;
      s_bias[i] = d < 0 || d >= p.window ? -INFINITY
                  : p.bias ? p.bias[head * p.bias_stride + min(d, p.distances - 1)] * 1.4426950408889634f : 0.f;
    }

  if (tid == 0) {
    tc::mbar_init(bar(LB_Q), 1);
    for (int s = 0; s < 2; ++s) {
      tc::mbar_init(bar(LB_KFULL + s), 1);
      tc::mbar_init(bar(LB_KEMPTY + s), 1);
      tc::mbar_init(bar(LB_VFULL + s), 1);
      tc::mbar_init(bar(LB_VEMPTY + s), 1);
      tc::mbar_init(bar(LB_SFULL + s), 1);
      tc::mbar_init(bar(LB_PREADY + s), 128);
      tc::mbar_init(bar(LB_ODONE + s), 1);
    }
    tc::mbar_init(bar(LB_DRAIN), 1);
    tc::mbar_fence_init();
  }
  if (warp == 8) {
    tc::tmem_alloc(smem_u32(&s_tmem), 512);
    tc::tmem_relinquish();
  }
  tc::fence_before_sync();
  __syncthreads();
  tc::fence_after_sync();
  const uint32_t tmem = s_tmem;

  if (warp >= 8) {
    tc::setmaxnreg_dec_40();
    if (warp == 8) {
      if (lane == 0) {
        const int tiles = n_b > 0 ? 2 : 1;
        tc::mbar_expect_tx(bar(LB_Q), tiles * Sh::kQBytes);
        for (int t = 0; t < tiles; ++t)
          for (int b = 0; b < NQ; ++b) {
            const uint32_t dst = q_smem + t * Sh::kQBytes + b * kLfBox;
            const int row = q_start + q0 + t * kSecond;
            if (kDiff) tc::tma_load_3d(dst, &tm_qn, 64 * b, 2 * head + t, row, bar(LB_Q));
            else if (b < p.nd) tc::tma_load_3d(dst, &tm_qn, 64 * b, head, row, bar(LB_Q));
            else tc::tma_load_3d(dst, &tm_qr, 64 * (b - p.nd), head, row, bar(LB_Q));
          }
        for (int i = 0; i < n_kv - lo_a; ++i) {
          const int s = i % KS, row = k_start + (lo_a + i) * kLfTile;
          tc::mbar_wait(bar(LB_KEMPTY + s), ((i / KS) & 1) ^ 1, abort_flag, p.error_word, 1);
          tc::mbar_expect_tx(bar(LB_KFULL + s), Sh::kKBytes);
          for (int b = 0; b < Sh::kKBytes / kLfBox; ++b) {
            const uint32_t dst = k_smem + s * Sh::kKBytes + b * kLfBox;
            if (kDiff) tc::tma_load_3d(dst, &tm_kn, 64 * (b % NQ), 2 * kv_head + b / NQ, row, bar(LB_KFULL + s));
            else if (b < p.nd) tc::tma_load_3d(dst, &tm_kn, 64 * b, kv_head, row, bar(LB_KFULL + s));
            else tc::tma_load_3d(dst, &tm_kr, 64 * (b - p.nd), 0, row, bar(LB_KFULL + s));
          }
          const int vs = i % VS;
          tc::mbar_wait(bar(LB_VEMPTY + vs), ((i / VS) & 1) ^ 1, abort_flag, p.error_word, 2);
          tc::mbar_expect_tx(bar(LB_VFULL + vs), Sh::kVBytes);
          for (int b = 0; b < NV; ++b)
            tc::tma_load_3d(v_smem + vs * Sh::kVBytes + b * kLfBox, &tm_v, 64 * b, kv_head, row, bar(LB_VFULL + vs));
        }
        if (*abort_flag) {       // copies in flight must land before the shared memory goes away
          tc::mbar_wait_timed(bar(LB_Q), 0);
          const int n = n_kv - lo_a;
          for (int i = max(n - 2, 0); i < n; ++i) {
            if (i >= n - KS) tc::mbar_wait_timed(bar(LB_KFULL + i % KS), (i / KS) & 1);
            if (i >= n - VS) tc::mbar_wait_timed(bar(LB_VFULL + i % VS), (i / VS) & 1);
          }
        }
      }
    } else if (warp == 9) {
      const uint32_t idesc_qk = tc::instr_desc_f16(1, 1, false, 128, 128);
      const uint32_t idesc_pv = tc::instr_desc_f16(1, 1, true, 128, 64 * NV);
      const uint32_t q_lo = tc::desc_lo(q_smem, 16), k_lo = tc::desc_lo(k_smem, 16), v_lo = tc::desc_lo(v_smem, kLfBox);
      auto issue_qk = [&](int t, int s) {
#pragma unroll
        for (int b = 0; b < NQ; ++b)
          tc::mma_ss_k64(tmem + t * 128, tc::desc64(q_lo + ((t * Sh::kQBytes + b * kLfBox) >> 4), tc::kDescHiSw128Sbo1024),
                         tc::desc64(k_lo + ((s * Sh::kKBytes + (kDiff ? t * Sh::kQBytes : 0) + b * kLfBox) >> 4), tc::kDescHiSw128Sbo1024), idesc_qk, b > 0);
        tc::commit_elected(bar(LB_SFULL + t), 0, false);
      };
      tc::mbar_wait(bar(LB_Q), 0, abort_flag, p.error_word, 3);
      tc::mbar_wait(bar(LB_KFULL + 0), 0, abort_flag, p.error_word, 4);
      tc::fence_after_sync();
      __syncwarp();
      issue_qk(0, 0);
      if (n_b > 0 && lo_b == lo_a) issue_qk(1, 0);
      tc::commit_elected(bar(LB_KEMPTY + 0), 0, false);
      for (int j = lo_a; j < n_kv; ++j) {
        const int i = j - lo_a, vs = i % VS, s1 = (i + 1) % KS;
        const bool more = j + 1 < n_kv;
        tc::mbar_wait(bar(LB_VFULL + vs), (i / VS) & 1, abort_flag, p.error_word, 5);
        if (more) tc::mbar_wait(bar(LB_KFULL + s1), ((i + 1) / KS) & 1, abort_flag, p.error_word, 6);
        for (int t = 0; t < 2; ++t) {
          const int n_t = t == 0 ? n_a : n_b, lo_t = t == 0 ? lo_a : lo_b;
          if (j >= lo_t && j < n_t) {
            tc::mbar_wait(bar(LB_PREADY + t), (j - lo_t) & 1, abort_flag, p.error_word, 7);
            tc::fence_after_sync();
            __syncwarp();
            tc::mma_ts_k128_commit(tmem + 256 + t * 128, tmem + t * 128,
                                   tc::desc64(v_lo + ((vs * Sh::kVBytes) >> 4), tc::kDescHiSw128Sbo1024), idesc_pv,
                                   j > lo_t, bar(LB_ODONE + t));
          }
          if (j + 1 >= lo_t && j + 1 < n_t) {
            if (kWin) {        // the first product of a query tile whose window opens here
              tc::fence_after_sync();
              __syncwarp();
            }
            issue_qk(t, s1);
          }
        }
        tc::commit_elected(bar(LB_VEMPTY + vs), bar(LB_KEMPTY + s1), more);
      }
      if (*abort_flag) {
        __syncwarp();
        tc::commit_elected(bar(LB_DRAIN), 0, false);
        tc::mbar_wait_timed(bar(LB_DRAIN), 0);
      }
    }
  } else {
    tc::setmaxnreg_inc_232();
    const int t = warp >> 2, n_t = t == 0 ? n_a : n_b, lo_t = t == 0 ? lo_a : lo_b;
    if (n_t > 0) {
      const int row = (warp & 3) * 32 + lane;
      const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
      const uint32_t s_addr = tmem + lane_addr + t * 128, o_addr = tmem + lane_addr + 256 + t * 128;
      const int low = kDiff ? (first_pos + row) / p.chunk * p.chunk : 0;      // first key of the row's chunk
      float m_used = -INFINITY, l = 0.f;
      for (int j = lo_t; j < n_t; ++j) {
        tc::mbar_wait(bar(LB_SFULL + t), (j - lo_t) & 1, abort_flag, p.error_word, 8);
        tc::fence_after_sync();
        // key 128j + col is visible to this row when col <= vis
        const int vis = first_pos + t * kSecond + row - j * kLfTile;
        uint32_t sv[4][32];
#pragma unroll
        for (int c = 0; c < 4; ++c) tc::tmem_ld32(s_addr + c * 32, sv[c]);
        tc::wait_ld();
        if constexpr (kWin) {
          const int d0 = first_pos + t * kLfTile - j * kLfTile;        // distance of the first row to the first key
          if (d0 - (kLfTile - 1) < p.distances - 1) {
            const float* tab = s_bias + kLfBefore + vis;
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
              for (int i = 0; i < 32; ++i)
                sv[c][i] = __float_as_uint(fmaf(__uint_as_float(sv[c][i]), p.scale_log2, tab[-(c * 32 + i)]));
          } else {
            const float far = s_bias[kLfBefore + p.distances - 1];
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
              for (int i = 0; i < 32; ++i) sv[c][i] = __float_as_uint(fmaf(__uint_as_float(sv[c][i]), p.scale_log2, far));
            if (d0 + kLfTile - 1 >= p.window) {                        // keys in front of the last row's window
#pragma unroll
              for (int c = 0; c < 4; ++c)
#pragma unroll
                for (int i = 0; i < 32; ++i)
                  if (vis - (c * 32 + i) >= p.window) sv[c][i] = 0xff800000u;
            }
          }
        } else if (kDiff) {
          // the tile reaches past the first row's position, or begins in front of the last row's chunk
          if (first_pos - j * kLfTile < kLfTile - 1 || (first_pos + kLfTile - 1) / p.chunk * p.chunk > j * kLfTile) {
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
              for (int i = 0; i < 32; ++i)
                if (c * 32 + i > vis || c * 32 + i < low - j * kLfTile) sv[c][i] = 0xff800000u;
          }
        } else if (first_pos + t * kLfTile - j * kLfTile < kLfTile - 1) {     // the tile reaches past the first row's position
#pragma unroll
          for (int c = 0; c < 4; ++c)
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (c * 32 + i > vis) sv[c][i] = 0xff800000u;
        }
        float mxs[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) mxs[i] = -INFINITY;
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 16; ++i)
            mxs[i & 7] = tc::max3(mxs[i & 7], __uint_as_float(sv[c][2 * i]), __uint_as_float(sv[c][2 * i + 1]));
        float mx = fmaxf(tc::max3(mxs[0], mxs[1], mxs[2]), tc::max3(mxs[3], mxs[4], mxs[5]));
        mx = tc::max3(mx, mxs[6], mxs[7]);
        if (!kWin) mx *= p.scale_log2;
        const bool grow = mx > m_used + kLfRescale;
        if (j > lo_t && __any_sync(0xffffffffu, grow)) {    // rare: move the reference maximum, rescale O
          const float alpha = grow ? fast_exp2(m_used - mx) : 1.f;      // 0 while nothing was visible
          tc::mbar_wait(bar(LB_ODONE + t), (j - lo_t - 1) & 1, abort_flag, p.error_word, 9);
          tc::fence_after_sync();
#pragma unroll 1
          for (int c = 0; c < 2 * NV; ++c) {
            uint32_t ov[32];
            tc::tmem_ld32(o_addr + c * 32, ov);
            tc::wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * alpha);
            tc::tmem_st32(o_addr + c * 32, ov);
          }
          tc::wait_st();
          l *= alpha;
        }
        if (grow) m_used = mx;
        const float off = FORM != LF_LATENT && m_used == -INFINITY ? 0.f : -m_used;         // a tile in front of the row's window or chunk
        const float2 sc2 = make_float2(p.scale_log2, p.scale_log2), nm2 = make_float2(off, off);
        float2 sums[4] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
        for (int c2 = 0; c2 < 2; ++c2) {
          uint32_t pk[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int c = 2 * c2 + (i >> 4), k = (i & 15) * 2;
            const float2 s2 = make_float2(__uint_as_float(sv[c][k]), __uint_as_float(sv[c][k + 1]));
            const float2 x = kWin ? tc::add2(s2, nm2) : tc::fma2(s2, sc2, nm2);
            float2 e;
            if ((i & 3) == 3) {
              e = tc::ex2_poly2(x);
            } else {
              e.x = tc::ex2_mufu(x.x);
              e.y = tc::ex2_mufu(x.y);
            }
            sums[i & 3] = tc::add2(sums[i & 3], e);
            pk[i] = pack2<__nv_bfloat16>(e.x, e.y);
          }
          tc::tmem_st32(s_addr + c2 * 32, pk);
        }
        const float2 s01 = tc::add2(sums[0], sums[1]), s23 = tc::add2(sums[2], sums[3]);
        l += (s01.x + s01.y) + (s23.x + s23.y);
        tc::wait_st();
        tc::fence_before_sync();
        tc::mbar_arrive(bar(LB_PREADY + t));
      }
      tc::mbar_wait(bar(LB_ODONE + t), (n_t - lo_t - 1) & 1, abort_flag, p.error_word, 10);
      tc::fence_after_sync();
      if constexpr (kDiff) {
        // queries are no longer wanted: [problem][row] factors, then [group][row] sums of squares take their place
        float* s_f = reinterpret_cast<float*>(smem_raw + (q_smem - smem_u32(smem_raw)));
        auto slot = [&](int u) -> float& { return s_f[u * (Sh::kQBytes / 4) + row]; };
        slot(t) = l > 0.f ? (t ? p.lambda : 1.f) / l : 0.f;
        tc::fence_before_sync();
        asm volatile("bar.sync 1, 256;" ::: "memory");
        tc::fence_after_sync();
        const float f1 = slot(0), f2 = slot(1);
        const uint32_t o1 = tmem + lane_addr + 256 + t * 32 * NV, o2 = o1 + 128;
        float o[NV][32], sq = 0.f;
#pragma unroll
        for (int c = 0; c < NV; ++c) {
          uint32_t u[32], v[32];
          tc::tmem_ld32(o1 + c * 32, u);
          tc::tmem_ld32(o2 + c * 32, v);
          tc::wait_ld();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            o[c][i] = __uint_as_float(u[i]) * f1 - __uint_as_float(v[i]) * f2;
            sq = fmaf(o[c][i], o[c][i], sq);       // columns past vdim are zero
          }
        }
        float* s_sq = s_f + kLfTile;
        s_sq[t * (Sh::kQBytes / 4) + row] = sq;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        sq = s_sq[row] + s_sq[Sh::kQBytes / 4 + row];
        const float f = p.mult / sqrtf(sq / static_cast<float>(p.vdim) + p.eps);
        if (q0 + row < q_len) {
          const int64_t tok = q_start + q0 + row;
          const __nv_bfloat16* gate = p.gate + tok * p.gate_stride + static_cast<int64_t>(head) * p.vdim;
          __nv_bfloat16* orow = p.out + tok * p.out_stride + static_cast<int64_t>(head) * p.vdim;
#pragma unroll
          for (int c = 0; c < NV; ++c)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const int d = (t * NV + c) * 32 + i * 8;
              if (d >= p.vdim) continue;
              float g[8];
              Vec<__nv_bfloat16, 8>::load(gate + d, g);
#pragma unroll
              for (int e = 0; e < 8; ++e) g[e] = o[c][8 * i + e] * f * sigmoid_t<__nv_bfloat16>(g[e]);
              Vec<__nv_bfloat16, 8>::store(orow + d, g);
            }
        }
      } else {
      float f = 1.f;
      if (p.sink) {
        const float sk = __bfloat162float(p.sink[head]) * 1.4426950408889634f, mm = fmaxf(m_used, sk);
        f = exp2f(m_used - mm);
        l = l * f + exp2f(sk - mm);
      }
      const float inv = l > 0.f ? f / l : 0.f;
      const int qrow = q0 + t * kLfTile + row;
      __nv_bfloat16* orow = p.out + static_cast<int64_t>(q_start + qrow) * p.out_stride + static_cast<int64_t>(head) * p.vdim;
      const bool turn = kWin && p.turn && qrow < q_len;
      const float2* angle = p.turn;      // neighbouring rows read neighbouring entries
      if (turn) angle += min(max(p.positions[q_start + qrow], static_cast<int64_t>(0)), p.table_rows - 1);
#pragma unroll
      for (int c = 0; c < 2 * NV; ++c) {
        uint32_t ov[32];
        tc::tmem_ld32(o_addr + c * 32, ov);
        tc::wait_ld();
        if (qrow < q_len) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if (c * 32 + i * 8 >= p.vdim) continue;
            if (turn) {
#pragma unroll
              for (int e = 0; e < 4; ++e)
                turn_back(ov[8 * i + 2 * e], ov[8 * i + 2 * e + 1], __ldg(angle + (c * 16 + i * 4 + e) * p.table_rows));
            }
            uint4 w;
            w.x = pack2<__nv_bfloat16>(__uint_as_float(ov[8 * i + 0]) * inv, __uint_as_float(ov[8 * i + 1]) * inv);
            w.y = pack2<__nv_bfloat16>(__uint_as_float(ov[8 * i + 2]) * inv, __uint_as_float(ov[8 * i + 3]) * inv);
            w.z = pack2<__nv_bfloat16>(__uint_as_float(ov[8 * i + 4]) * inv, __uint_as_float(ov[8 * i + 5]) * inv);
            w.w = pack2<__nv_bfloat16>(__uint_as_float(ov[8 * i + 6]) * inv, __uint_as_float(ov[8 * i + 7]) * inv);
            st_global16(orow + c * 32 + i * 8, w);
          }
        }
      }
      }
    }
  }
  __syncwarp();
  tc::fence_before_sync();
  __syncthreads();
  if (warp == 8) {
    tc::fence_after_sync();
    tc::tmem_dealloc(tmem, 512);
  }
}

// Rows of the paged cache of every sequence, packed: out[cu_k[s] + j] = cache row of position first[s] + j of sequence s
// (first null: 0).  Rows without a block read as zero.
__global__ void __launch_bounds__(256)
latent_gather_kernel(uint4* __restrict__ out, const uint4* __restrict__ cache, const int32_t* __restrict__ cu_k,
                     const int32_t* __restrict__ first, int num_seqs, int64_t keys, const int32_t* __restrict__ tables, int64_t bt_stride, int max_blocks,
                     int block_size, int64_t num_blocks, int chunks) {
  const int lane = threadIdx.x & 31;
  for (int64_t r = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5); r < keys; r += static_cast<int64_t>(gridDim.x) * 8) {
    const int s = seq_of_token(cu_k, num_seqs, static_cast<int>(r));
    const int pos = static_cast<int>(r) - cu_k[s] + (first ? first[s] : 0), blk = pos / block_size;
    const int32_t phys = blk < max_blocks ? tables[static_cast<int64_t>(s) * bt_stride + blk] : -1;
    const bool ok = phys >= 0 && phys < num_blocks;
    const int64_t src = ok ? (static_cast<int64_t>(phys) * block_size + (pos - blk * block_size)) * chunks : 0;
    for (int c = lane; c < chunks; c += 32) out[r * chunks + c] = ok ? cache[src + c] : make_uint4(0, 0, 0, 0);
  }
}

template <int NQ, int NV, int FORM = LF_LATENT>
static int launch_latent_prefill(const CUtensorMap (&tm)[5], const LfParams& p, int64_t tokens, int heads, cudaStream_t st) {
  using Sh = LfShape<NQ, NV, FORM>;
  constexpr bool kWin = FORM == LF_WINDOW;
  constexpr int kRows = FORM == LF_DIFF ? kLfTile : 2 * kLfTile;
  const char* what = kWin ? "window_prefill" : FORM == LF_DIFF ? "diff_prefill" : "latent_prefill";
  int smem = Sh::kSmem;
  if (kWin) {
    const int table = kLfBefore + p.distances + kLfAfter;
    if (table > Sh::kTable) return fail(MV_ERR_LIMIT, "window_prefill: %d distances (at most %d)", p.distances, Sh::kTable - kLfBefore - kLfAfter);
    smem += table * 4;
  }
  const cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel<NQ, NV, FORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return fail(MV_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
  const dim3 grid(static_cast<unsigned>(tokens / kRows + std::min<int64_t>(p.num_seqs, tokens)), heads);
  latent_prefill_kernel<NQ, NV, FORM><<<grid, kLfThreads, smem, st>>>(tm[0], tm[1], tm[2], tm[3], tm[4], p);
  return check_launch(what);
}

}  // namespace mv

extern "C" int mv_latent_gather(void* out, const void* cache, const int32_t* cu_k, const int32_t* first, int num_seqs,
                                int64_t keys, const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size,
                                int64_t num_blocks, int row, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "latent_gather: dtype %d", dtype);
  const int bytes = row * (dtype == MV_F32 ? 4 : 2);
  if (keys < 0 || num_seqs < 0 || block_size <= 0 || row <= 0 || bytes % 16) return fail(MV_ERR_SHAPE, "latent_gather: row %d", row);
  if (keys == 0 || num_seqs == 0) return MV_OK;
  if (!out || !cache || !cu_k || !block_tables) return fail(MV_ERR_NULL, "latent_gather: null pointer");
  if (!aligned16(out) || !aligned16(cache)) return fail(MV_ERR_ALIGN, "latent_gather: alignment");
  const unsigned grid = static_cast<unsigned>(std::min<int64_t>((keys + 7) / 8, kNumSMs * 16));
  latent_gather_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<uint4*>(out), static_cast<const uint4*>(cache), cu_k, first, num_seqs, keys, block_tables, bt_stride, max_blocks, block_size,
      num_blocks, bytes / 16);
  return check_launch("latent_gather");
}

extern "C" int mv_latent_prefill(void* out, int64_t out_stride, const void* q, int64_t q_stride, const void* k,
                                 int64_t k_stride, const void* k_rot, int64_t k_rot_stride, const void* v,
                                 int64_t v_stride, const int32_t* cu_q, const int32_t* cu_k, int num_seqs,
                                 int64_t tokens, int64_t keys, int heads, int dim, int rot_dim, int vdim, float scale,
                                 const void* sink, int* error_word, void* stream) {
  using namespace mv;
  if (num_seqs < 0 || tokens < 0 || keys < tokens || heads <= 0 || dim <= 0 || rot_dim < 0 || vdim <= 0 || !(scale > 0.f))
    return fail(MV_ERR_SHAPE, "latent_prefill: heads %d dim %d rot_dim %d vdim %d", heads, dim, rot_dim, vdim);
  const int nd = (dim + 63) / 64, nq = nd + (rot_dim + 63) / 64, nv = (vdim + 63) / 64;
  if (dim % 8 || rot_dim % 8 || vdim % 8 || nq > 3 || nv > 2)
    return fail(MV_ERR_LIMIT, "latent_prefill: dim %d rot_dim %d vdim %d", dim, rot_dim, vdim);
  if (tokens == 0 || num_seqs == 0) return MV_OK;
  if (!out || !q || !k || (rot_dim && !k_rot) || !v || !cu_q || !cu_k || !error_word) return fail(MV_ERR_NULL, "latent_prefill: null pointer");
  if (!vec8_ok(out, out_stride, 2) || !vec8_ok(q, q_stride, 2) || !vec8_ok(k, k_stride, 2) || !vec8_ok(k_rot, k_rot_stride, 2) ||
      !vec8_ok(v, v_stride, 2))
    return fail(MV_ERR_ALIGN, "latent_prefill: rows must start on 16-byte boundaries");
  const char* w = "latent_prefill";
  CUtensorMap tm[5];
  const auto* qb = static_cast<const __nv_bfloat16*>(q);
  int rc = make_tmap_bf16(&tm[0], q, dim, heads, tokens, dim + rot_dim, q_stride, 1, kLfTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[2], k, dim, heads, keys, dim, k_stride, 1, kLfTile, w);
  if (!rc && rot_dim) rc = make_tmap_bf16(&tm[1], qb + dim, rot_dim, heads, tokens, dim + rot_dim, q_stride, 1, kLfTile, w);
  if (!rc && rot_dim) rc = make_tmap_bf16(&tm[3], k_rot, rot_dim, 1, keys, rot_dim, k_rot_stride, 1, kLfTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[4], v, vdim, heads, keys, vdim, v_stride, 1, kLfTile, w);
  if (rc) return rc;
  if (!rot_dim) { tm[1] = tm[0]; tm[3] = tm[2]; }
  LfParams p{static_cast<__nv_bfloat16*>(out), out_stride, vdim, cu_q, cu_k, num_seqs, nd, dim, rot_dim,
             scale * 1.4426950408889634f, static_cast<const __nv_bfloat16*>(sink), error_word, 1, 0, 0, nullptr, 0, nullptr, 0, nullptr, 1, nullptr, 0, 0.f, 0.f, 0.f};
  auto st = static_cast<cudaStream_t>(stream);
  if (nq == 1) return nv == 1 ? launch_latent_prefill<1, 1>(tm, p, tokens, heads, st) : launch_latent_prefill<1, 2>(tm, p, tokens, heads, st);
  if (nq == 2) return nv == 1 ? launch_latent_prefill<2, 1>(tm, p, tokens, heads, st) : launch_latent_prefill<2, 2>(tm, p, tokens, heads, st);
  return nv == 1 ? launch_latent_prefill<3, 1>(tm, p, tokens, heads, st) : launch_latent_prefill<3, 2>(tm, p, tokens, heads, st);
}

// Distances of the bias table that the kernel takes at these sizes, or -1 when it does not take them.
extern "C" int mv_window_prefill_distances(int dim, int vdim) {
  using namespace mv;
  if (dim <= 0 || vdim <= 0 || dim % 8 || vdim % 8 || dim > 192 || vdim > 128) return -1;
  const int nq = (dim + 63) / 64, extra = kLfBefore + kLfAfter;
  if (nq == 1) return (vdim <= 64 ? LfShape<1, 1, LF_WINDOW>::kTable : LfShape<1, 2, LF_WINDOW>::kTable) - extra;
  if (nq == 2) return (vdim <= 64 ? LfShape<2, 1, LF_WINDOW>::kTable : LfShape<2, 2, LF_WINDOW>::kTable) - extra;
  return (vdim <= 64 ? LfShape<3, 1, LF_WINDOW>::kTable : LfShape<3, 2, LF_WINDOW>::kTable) - extra;
}

extern "C" int mv_window_prefill(void* out, int64_t out_stride, const void* q, int64_t q_stride, const void* k,
                                 int64_t k_stride, const void* v, int64_t v_stride, const int32_t* cu_q,
                                 const int32_t* cu_k, int num_seqs, int64_t tokens, int64_t keys, int heads, int kv_heads,
                                 int dim, int vdim, int64_t window, float scale, const float* bias, int64_t bias_stride,
                                 int distances, const void* sink, const float* turn, int64_t table_rows,
                                 const int64_t* positions, int* error_word, void* stream) {
  using namespace mv;
  const char* w = "window_prefill";
  if (num_seqs < 0 || tokens < 0 || keys < tokens || heads <= 0 || kv_heads <= 0 || heads % kv_heads || window <= 0 || distances <= 0)
    return fail(MV_ERR_SHAPE, "window_prefill: heads %d over %d, window %lld, %d distances", heads, kv_heads, static_cast<long long>(window), distances);
  if (turn && (table_rows <= 0 || !positions || (reinterpret_cast<uintptr_t>(turn) & 7u)))
    return fail(MV_ERR_NULL, "window_prefill: rotation table");
  if (mv_window_prefill_distances(dim, vdim) < 0) return fail(MV_ERR_LIMIT, "window_prefill: dim %d vdim %d", dim, vdim);
  if (tokens == 0 || num_seqs == 0) return MV_OK;
  if (!out || !q || !k || !v || !cu_q || !cu_k || !error_word) return fail(MV_ERR_NULL, "window_prefill: null pointer");
  if (!vec8_ok(out, out_stride, 2) || !vec8_ok(q, q_stride, 2) || !vec8_ok(k, k_stride, 2) || !vec8_ok(v, v_stride, 2))
    return fail(MV_ERR_ALIGN, "window_prefill: rows must start on 16-byte boundaries");
  CUtensorMap tm[5];
  int rc = make_tmap_bf16(&tm[0], q, dim, heads, tokens, dim, q_stride, 1, kLfTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[2], k, dim, kv_heads, keys, dim, k_stride, 1, kLfTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[4], v, vdim, kv_heads, keys, vdim, v_stride, 1, kLfTile, w);
  if (rc) return rc;
  tm[1] = tm[0];
  tm[3] = tm[2];
  const int nq = (dim + 63) / 64, nv = (vdim + 63) / 64;
  const int win = static_cast<int>(std::min<int64_t>(window, 1 << 30));
  LfParams p{static_cast<__nv_bfloat16*>(out), out_stride, vdim, cu_q, cu_k, num_seqs, nq, dim, 0,
             scale * 1.4426950408889634f, static_cast<const __nv_bfloat16*>(sink), error_word, heads / kv_heads, win,
             bias ? std::min(distances, win) : 1, bias, bias_stride, reinterpret_cast<const float2*>(turn), table_rows, positions,
             1, nullptr, 0, 0.f, 0.f, 0.f};
  auto st = static_cast<cudaStream_t>(stream);
  if (nq == 1) return nv == 1 ? launch_latent_prefill<1, 1, LF_WINDOW>(tm, p, tokens, heads, st) : launch_latent_prefill<1, 2, LF_WINDOW>(tm, p, tokens, heads, st);
  if (nq == 2) return nv == 1 ? launch_latent_prefill<2, 1, LF_WINDOW>(tm, p, tokens, heads, st) : launch_latent_prefill<2, 2, LF_WINDOW>(tm, p, tokens, heads, st);
  return nv == 1 ? launch_latent_prefill<3, 1, LF_WINDOW>(tm, p, tokens, heads, st) : launch_latent_prefill<3, 2, LF_WINDOW>(tm, p, tokens, heads, st);
}

extern "C" int mv_diff_prefill_takes(int dim, int vdim) {
  return dim > 0 && vdim > 0 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 128 && vdim <= 128;
}

extern "C" int mv_diff_prefill(void* out, const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v,
                               int64_t v_stride, const int32_t* cu_q, const int32_t* cu_k, int num_seqs, int64_t tokens,
                               int64_t keys, int64_t chunk, const void* gate, int64_t gate_stride, float lambda, float mult,
                               float eps, int heads, int kv_heads, int dim, int vdim, float scale, int* error_word,
                               void* stream) {
  using namespace mv;
  const char* w = "diff_prefill";
  if (num_seqs < 0 || tokens < 0 || keys < tokens || heads <= 0 || kv_heads <= 0 || heads % kv_heads || chunk <= 0 || !(scale > 0.f))
    return fail(MV_ERR_SHAPE, "diff_prefill: heads %d over %d, chunk %lld, scale %f", heads, kv_heads, static_cast<long long>(chunk), scale);
  if (!mv_diff_prefill_takes(dim, vdim)) return fail(MV_ERR_LIMIT, "diff_prefill: dim %d vdim %d", dim, vdim);
  if (tokens == 0 || num_seqs == 0) return MV_OK;
  if (!out || !q || !k || !v || !cu_q || !cu_k || !gate || !error_word) return fail(MV_ERR_NULL, "diff_prefill: null pointer");
  if (!aligned16(out) || !vec8_ok(q, q_stride, 2) || !vec8_ok(k, k_stride, 2) || !vec8_ok(v, v_stride, 2) || !vec8_ok(gate, gate_stride, 2))
    return fail(MV_ERR_ALIGN, "diff_prefill: rows must start on 16-byte boundaries");
  CUtensorMap tm[5];
  int rc = make_tmap_bf16(&tm[0], q, dim, 2 * heads, tokens, dim, q_stride, 1, kLfTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[2], k, dim, 2 * kv_heads, keys, dim, k_stride, 1, kLfTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[4], v, vdim, kv_heads, keys, vdim, v_stride, 1, kLfTile, w);
  if (rc) return rc;
  tm[1] = tm[0];
  tm[3] = tm[2];
  const int nq = (dim + 63) / 64, nv = (vdim + 63) / 64;
  LfParams p{static_cast<__nv_bfloat16*>(out), static_cast<int64_t>(heads) * vdim, vdim, cu_q, cu_k, num_seqs, nq, dim, 0,
             scale * 1.4426950408889634f, nullptr, error_word, heads / kv_heads, 1, 1, nullptr, 0, nullptr, 0, nullptr,
             static_cast<int>(std::min<int64_t>(chunk, 1 << 30)), static_cast<const __nv_bfloat16*>(gate), gate_stride, lambda, mult, eps};
  auto st = static_cast<cudaStream_t>(stream);
  if (nq == 1) return nv == 1 ? launch_latent_prefill<1, 1, LF_DIFF>(tm, p, tokens, heads, st) : launch_latent_prefill<1, 2, LF_DIFF>(tm, p, tokens, heads, st);
  return nv == 1 ? launch_latent_prefill<2, 1, LF_DIFF>(tm, p, tokens, heads, st) : launch_latent_prefill<2, 2, LF_DIFF>(tm, p, tokens, heads, st);
}
