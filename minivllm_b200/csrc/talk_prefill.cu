// Prefill of talking-heads attention (talk_attention.cu) on the Blackwell tensor cores, causal, packed batch.  The mixture of the
// heads' weights is linear, so that it can be taken after the weights have met the values: a CTA forms the weights of ONE head for
// 128 queries and applies them to the values of several value heads, up to 256 columns; head_mix_kernel combines the results.
//
// Scores are capped, so weights are formed against a fixed reference (TalkScore): no running maximum, no rescaling.  Two pairs of
// warpgroups take turns at the key tiles of the same queries, each warpgroup with 64 of a tile's 128 keys.
//   warps 0-15  weights (thread = row = TMEM lane); the bias of a tile's 255 distances, with -inf behind the query, is put into
//               shared memory while the tile's product is awaited
//   warp 16     TMA producer, warp 17 MMA issuer (S = Q K^T into two buffers, O += P V with P in TMEM, in two halves)
// The CTAs are persistent, one per SM: a unit is a tile of queries, a head and a run of value heads; the next unit's queries, keys
// and first scores are on their way while a unit's results are written.
// Tensor memory: S of pair b in columns 128 b .., P of a half where its S was, O in 256-511.
//
// Per weight: a power of two and a quarter of a reciprocal for the cap (one serves four keys), and an outer power of two, three
// eighths of which run on the FMA pipe, against 2 (dim + columns) tensor FLOPs: bound by the special-function unit and
// instruction issue.
#include <algorithm>
#include "mma.cuh"
#include "query_tile.cuh"
#include "talk.cuh"
#include "tcgen05.cuh"
#include "tmap.cuh"
#include "vec.cuh"

namespace mv {

constexpr int kTpThreads = 640, kTpTile = 128, kTpBox = kTpTile * 128;      // kTpBox: one 64-column box of a tile
constexpr int kTpTable = 2 * kTpTile;                 // distances of a tile
constexpr int kTpSeqs = 1024;                         // sequences whose bounds are kept in shared memory

struct TalkPrefillParams {
  __nv_bfloat16* out;                                 // (tokens, heads, kv_heads, vdim)
  const int32_t *cu_q, *cu_k;
  int num_seqs, heads, kv_heads, vdim;
  int boxes, per;                                     // 64-column boxes of a value head; value heads per CTA
  const float *r1, *r2;
  float scale, cap;
  int* error_word;
};

enum { TB_QFULL = 0, TB_QEMPTY = 1, TB_KFULL = 2, TB_KEMPTY = 4, TB_VFULL = 6, TB_VEMPTY = 8, TB_SFULL = 10, TB_PREADY = 12, TB_ODONE = 14,
       TB_OEMPTY = 15, TB_DRAIN = 16, TB_COUNT = 17 };

__host__ __device__ constexpr int talk_prefill_kstages(int nq, int boxes) { return nq == 2 && boxes > 3 ? 1 : 2; }
inline int talk_prefill_smem(int nq, int boxes, int num_seqs) {
  return ((1 + talk_prefill_kstages(nq, boxes)) * nq + 2 * boxes) * kTpBox + (4 * kTpTable + 8 * kTpTile) * 4 + 1024 +
         (num_seqs <= kTpSeqs ? 2 * (num_seqs + 1) * 4 : 0);
}

__device__ __forceinline__ void group_barrier(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

// A unit of work, as every warp sees it.
struct TalkUnit {
  int q_start, q_len, k_start, q0, first_pos, n;      // n: key tiles up to the last row's position
  int head, kv_head, v0, boxes;
  __device__ __forceinline__ bool find(const TalkPrefillParams& p, const int32_t* cu_q, const int32_t* cu_k, int u) {
    const int chunks = (p.kv_heads + p.per - 1) / p.per, across = p.heads * chunks, x = u / across, y = u - x * across;
    int seq, tile;
    if (!find_query_tile_warp(cu_q, p.num_seqs, kTpTile, x, seq, tile)) return false;
    head = y / chunks;
    v0 = (y - head * chunks) * p.per;
    kv_head = head / (p.heads / p.kv_heads);
    boxes = min(p.per, p.kv_heads - v0) * p.boxes;
    q_start = cu_q[seq];
    q_len = cu_q[seq + 1] - q_start;
    k_start = cu_k[seq];
    q0 = tile * kTpTile;
    const int behind = cu_k[seq + 1] - k_start - q_len;
    first_pos = behind + q0;
    n = (behind + min(q0 + kTpTile, q_len) + kTpTile - 1) / kTpTile;
    return true;
  }
};

template <int NQ>
__global__ void __launch_bounds__(kTpThreads, 1)
talk_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                    const __grid_constant__ CUtensorMap tm_v, const TalkPrefillParams p) {
  constexpr int kQBytes = NQ * kTpBox;
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t bars[TB_COUNT];
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort, s_sticky, s_stop[2];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int all = p.per * p.boxes, KS = talk_prefill_kstages(NQ, all);
  const uint32_t q_smem = (smem_u32(smem_raw) + 1023u) & ~1023u;      // [box][128][128B]
  const uint32_t k_smem = q_smem + kQBytes;                           // [stage KS][box]
  const uint32_t v_smem = k_smem + KS * kQBytes;                      // [stage 2][box]
  float* s_bias = reinterpret_cast<float*>(smem_raw + (v_smem + 2 * all * kTpBox - smem_u32(smem_raw)));   // [pair][buffer][distance]
  float* s_sum = s_bias + 4 * kTpTable;                                       // [unit & 1][group][row]
  int32_t* s_cu = reinterpret_cast<int32_t*>(s_sum + 8 * kTpTile);
  const uint32_t bar0 = smem_u32(bars);
  auto bar = [&](int i) { return bar0 + 8u * i; };
  volatile int* abort_flag = &s_abort;
  if (tid == 0) {
    s_abort = 0;
    s_sticky = *reinterpret_cast<volatile int*>(p.error_word);
    tc::tma_prefetch_desc(&tm_q);
    tc::tma_prefetch_desc(&tm_k);
    tc::tma_prefetch_desc(&tm_v);
    for (int i = 0; i < TB_COUNT; ++i)
      tc::mbar_init(bar(i), i == TB_PREADY || i == TB_PREADY + 1 ? 256 : i == TB_OEMPTY ? 512 : 1);
    tc::mbar_fence_init();
  }
  const int32_t *cu_q = p.cu_q, *cu_k = p.cu_k;
  if (p.num_seqs <= kTpSeqs) {
    for (int i = tid; i <= p.num_seqs; i += kTpThreads) {
      s_cu[i] = p.cu_q[i];
      s_cu[p.num_seqs + 1 + i] = p.cu_k[i];
    }
    cu_q = s_cu;
    cu_k = s_cu + p.num_seqs + 1;
  }
  if (warp == 17) {
    tc::tmem_alloc(smem_u32(&s_tmem), 512);
    tc::tmem_relinquish();
  }
  tc::fence_before_sync();
  __syncthreads();
  tc::fence_after_sync();
  const uint32_t tmem = s_tmem;
  const bool idle = s_sticky != 0;            // an earlier wait ran out
  TalkUnit w;
  // `t` counts key tiles over all units: tile t uses pair t & 1, value stage t & 1 and key stage t % KS
  if (warp >= 16) {
    tc::setmaxnreg_dec_40();
    if (warp == 16 && !idle) {
      int t = 0, unit = 0;
      auto values = [&](int i) {              // of the unit's tile i, converged
        const int at = t + i, s = at & 1;
        tc::mbar_wait(bar(TB_VEMPTY + s), ((at >> 1) & 1) ^ 1, abort_flag, p.error_word, 2);
        __syncwarp();
        if (lane == 0) tc::mbar_expect_tx(bar(TB_VFULL + s), w.boxes * kTpBox);
        __syncwarp();
#pragma unroll
        for (int b = 0; b < 4; ++b)
          if (b < w.boxes)
            tc::tma_load_3d_elected(v_smem + (s * all + b) * kTpBox, &tm_v, 64 * (b % p.boxes), w.v0 + b / p.boxes, w.k_start + i * kTpTile, bar(TB_VFULL + s));
      };
      for (int u = blockIdx.x; !*abort_flag && w.find(p, cu_q, cu_k, u); u += gridDim.x, ++unit) {
        __syncwarp();
        tc::mbar_wait(bar(TB_QEMPTY), (unit & 1) ^ 1, abort_flag, p.error_word, 3);
        __syncwarp();
        if (lane == 0) tc::mbar_expect_tx(bar(TB_QFULL), kQBytes);
        __syncwarp();
#pragma unroll
        for (int b = 0; b < NQ; ++b) tc::tma_load_3d_elected(q_smem + b * kTpBox, &tm_q, 64 * b, w.head, w.q_start + w.q0, bar(TB_QFULL));
        for (int i = 0; i < w.n; ++i) {       // keys one tile ahead of values
          const int at = t + i, s = at % KS;
          tc::mbar_wait(bar(TB_KEMPTY + s), ((at / KS) & 1) ^ 1, abort_flag, p.error_word, 1);
          __syncwarp();
          if (lane == 0) tc::mbar_expect_tx(bar(TB_KFULL + s), kQBytes);
          __syncwarp();
#pragma unroll
          for (int b = 0; b < NQ; ++b)
            tc::tma_load_3d_elected(k_smem + s * kQBytes + b * kTpBox, &tm_k, 64 * b, w.kv_head, w.k_start + i * kTpTile, bar(TB_KFULL + s));
          if (i > 0) values(i - 1);
        }
        values(w.n - 1);
        t += w.n;
      }
      if (*abort_flag && unit > 0) {       // copies in flight must land before the shared memory goes away
        tc::mbar_wait_timed(bar(TB_QFULL), (unit & 1) ^ 1);
        for (int at = max(t - 2, 0); at < t; ++at) {
          tc::mbar_wait_timed(bar(TB_KFULL + at % KS), (at / KS) & 1);
          tc::mbar_wait_timed(bar(TB_VFULL + (at & 1)), (at >> 1) & 1);
        }
      }
    } else if (warp == 17 && !idle) {
      const uint32_t idesc_qk = tc::instr_desc_f16(1, 1, false, kTpTile, kTpTile);
      const uint32_t q_lo = tc::desc_lo(q_smem, 16), k_lo = tc::desc_lo(k_smem, 16), v_lo = tc::desc_lo(v_smem, kTpBox);
      int t = 0, unit = 0;
      auto scores = [&](int i) {           // of the unit's tile i, into its pair's buffer
        const int at = t + i, s = at % KS;
        tc::mbar_wait(bar(TB_KFULL + s), (at / KS) & 1, abort_flag, p.error_word, 4);
        tc::fence_after_sync();
        __syncwarp();
#pragma unroll
        for (int b = 0; b < NQ; ++b)
          tc::mma_ss_k64(tmem + (at & 1) * kTpTile, tc::desc64(q_lo + ((b * kTpBox) >> 4), tc::kDescHiSw128Sbo1024),
                         tc::desc64(k_lo + ((s * kQBytes + b * kTpBox) >> 4), tc::kDescHiSw128Sbo1024), idesc_qk, b > 0);
        tc::commit_elected(bar(TB_SFULL + (at & 1)), bar(TB_KEMPTY + s), true);
        if (i == w.n - 1) tc::commit_elected(bar(TB_QEMPTY), 0, false);
      };
      for (int u = blockIdx.x; !*abort_flag && w.find(p, cu_q, cu_k, u); u += gridDim.x, ++unit) {
        __syncwarp();
        const uint32_t idesc_pv = tc::instr_desc_f16(1, 1, true, kTpTile, 64 * w.boxes);
        tc::mbar_wait(bar(TB_QFULL), unit & 1, abort_flag, p.error_word, 3);
        scores(0);
        if (w.n > 1) scores(1);
        for (int i = 0; i < w.n; ++i) {
          const int at = t + i, b = at & 1;
          tc::mbar_wait(bar(TB_VFULL + b), (at >> 1) & 1, abort_flag, p.error_word, 5);
          tc::mbar_wait(bar(TB_PREADY + b), (at >> 1) & 1, abort_flag, p.error_word, 7);
          if (i == 0) tc::mbar_wait(bar(TB_OEMPTY), (unit & 1) ^ 1, abort_flag, p.error_word, 6);      // the last unit's results are out
          tc::fence_after_sync();
          __syncwarp();
          const uint32_t v_at = v_lo + ((b * all * kTpBox) >> 4), a = tmem + b * kTpTile;
          tc::mma_ts_k64(tmem + 256, a, tc::desc64(v_at, tc::kDescHiSw128Sbo1024), idesc_pv, i > 0);
          tc::mma_ts_k64(tmem + 256, a + 64, tc::desc64(v_at + ((64 * 128) >> 4), tc::kDescHiSw128Sbo1024), idesc_pv, true);
          tc::commit_elected(bar(TB_VEMPTY + b), bar(TB_ODONE), i == w.n - 1);
          if (i + 2 < w.n) scores(i + 2);
        }
        t += w.n;
      }
      __syncwarp();
      if (*abort_flag) {
        __syncwarp();
        tc::commit_elected(bar(TB_DRAIN), 0, false);
        tc::mbar_wait_timed(bar(TB_DRAIN), 0);
      }
    }
  } else {
    tc::setmaxnreg_inc_104();
    const int g = warp >> 2, pair = g >> 1, half = g & 1, row = (warp & 3) * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t s_addr = tmem + lane_addr + g * 64;
    const TalkScore score(p.scale, p.cap);
    const float2 in2 = make_float2(score.in, score.in), out2 = make_float2(score.out, score.out), one2 = make_float2(1.f, 1.f);
    int t = 0, unit = 0;
    for (int u = blockIdx.x; !idle && w.find(p, cu_q, cu_k, u); u += gridDim.x, ++unit) {
      const float r1 = __ldg(p.r1 + w.head), r2 = __ldg(p.r2 + w.head);
      float2 sums[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
      for (int i = (t & 1) ^ pair; i < w.n; i += 2) {
        const int k = (t + i) >> 1;          // tiles of this pair before this one
        float* tab = s_bias + (pair * 2 + (k & 1)) * kTpTable;
        {
          const int x = half * kTpTile + row, d = w.first_pos - i * kTpTile - (kTpTile - 1) + x;     // x 0: first row, last key
          tab[x] = d < 0 ? -INFINITY : score.bias(r1, r2, d);
        }
        group_barrier(2 + pair, 256);
        tc::mbar_wait(bar(TB_SFULL + pair), k & 1, abort_flag, p.error_word, 8);
        tc::fence_after_sync();
        const float* mine = tab + row + (kTpTile - 1) - half * 64;     // the bias of this group's key col is mine[-col]
        uint32_t sv[2][16];
        tc::tmem_ld16(s_addr, sv[0]);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          tc::wait_ld();
          if (c < 3) tc::tmem_ld16(s_addr + (c + 1) * 16, sv[(c + 1) & 1]);
          const uint32_t(&sc)[16] = sv[c & 1];
          uint32_t pk[8];
#pragma unroll
          for (int y = 0; y < 8; y += 4) {         // eight keys; one reciprocal serves four of them
            float2 d[4];
#pragma unroll
            for (int v = 0; v < 4; ++v) {
              const float2 z = mul_f32x2(make_float2(__uint_as_float(sc[2 * (y + v)]), __uint_as_float(sc[2 * (y + v) + 1])), in2);
              d[v] = tc::add2(make_float2(tc::ex2_mufu(fminf(z.x, 30.f)), tc::ex2_mufu(fminf(z.y, 30.f))), one2);
            }
            const float2 lo = mul_f32x2(d[0], d[1]), hi = mul_f32x2(d[2], d[3]), dd = mul_f32x2(lo, hi);
            const float2 r = mul_f32x2(make_float2(fast_rcp(dd.x), fast_rcp(dd.y)), out2), rl = mul_f32x2(r, hi), rh = mul_f32x2(r, lo);
#pragma unroll
            for (int v = 0; v < 4; ++v) {
              const int col = c * 16 + 2 * (y + v);
              const float2 x = tc::fma2(v < 2 ? rl : rh, d[v ^ 1], make_float2(mine[-col], mine[-col - 1]));
              float2 e;
              if (v == 3 || (v == 1 && y == 0)) {      // three of eight: both pipes are about equally busy
                e = tc::ex2_poly2(x);
              } else {
                e.x = tc::ex2_mufu(x.x);
                e.y = tc::ex2_mufu(x.y);
              }
              sums[v & 1] = tc::add2(sums[v & 1], e);
              pk[y + v] = pack2<__nv_bfloat16>(e.x, e.y);
            }
          }
          tc::tmem_st8(s_addr + c * 8, pk);
        }
        tc::wait_st();
        tc::fence_before_sync();
        tc::mbar_arrive(bar(TB_PREADY + pair));
      }
      t += w.n;
      const float2 both = tc::add2(sums[0], sums[1]);
      float* sum = s_sum + (unit & 1) * 4 * kTpTile;
      sum[g * kTpTile + row] = both.x + both.y;
      if (tid == 0) s_stop[unit & 1] = *abort_flag;
      group_barrier(1, 512);
      const bool stop = s_stop[unit & 1] != 0;
      float l = 0.f;
#pragma unroll
      for (int x = 0; x < 4; ++x) l += sum[x * kTpTile + row];
      const float inv = l > 0.f ? 1.f / l : 0.f;
      tc::mbar_wait(bar(TB_ODONE), unit & 1, abort_flag, p.error_word, 10);
      tc::fence_after_sync();
      const int qrow = w.q0 + row, vh = g / p.boxes, d0 = (g - vh * p.boxes) * 64;      // one box of 64 columns per group
      __nv_bfloat16* orow = p.out + ((static_cast<int64_t>(w.q_start + qrow) * p.heads + w.head) * p.kv_heads + w.v0 + vh) * p.vdim + d0;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t ov[32];
        if (g < w.boxes) {
          tc::tmem_ld32(tmem + lane_addr + 256 + g * 64 + c * 32, ov);
          tc::wait_ld();
        }
        if (c == 1) {
          tc::fence_before_sync();
          tc::mbar_arrive(bar(TB_OEMPTY));
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {      // 16 columns: a whole sector, when rows are whole sectors
          const int d = c * 32 + i * 16;
          if (g >= w.boxes || qrow >= w.q_len) continue;
          uint32_t x[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) x[e] = pack2<__nv_bfloat16>(__uint_as_float(ov[i * 16 + 2 * e]) * inv, __uint_as_float(ov[i * 16 + 2 * e + 1]) * inv);
          const uint4 lo = make_uint4(x[0], x[1], x[2], x[3]), hi = make_uint4(x[4], x[5], x[6], x[7]);
          if (p.vdim % 16 == 0) {
            if (d0 + d < p.vdim) st_global32(orow + d, lo, hi);
          } else {
            if (d0 + d < p.vdim) st_global16(orow + d, lo);
            if (d0 + d + 8 < p.vdim) st_global16(orow + d + 8, hi);
          }
        }
        __syncwarp();
      }
      if (stop) break;
    }
  }
  __syncwarp();
  tc::fence_before_sync();
  __syncthreads();
  if (warp == 17) {
    tc::fence_after_sync();
    tc::tmem_dealloc(tmem, 512);
  }
}

template <int NQ>
static int launch_talk_prefill(const CUtensorMap (&tm)[3], const TalkPrefillParams& p, int64_t tokens, cudaStream_t st) {
  const int smem = talk_prefill_smem(NQ, p.per * p.boxes, p.num_seqs);
  const cudaError_t e = cudaFuncSetAttribute(talk_prefill_kernel<NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return fail(MV_ERR_CUDA, "talk_prefill: %s", cudaGetErrorString(e));
  const int64_t units = (tokens / kTpTile + std::min<int64_t>(p.num_seqs, tokens)) * p.heads * ((p.kv_heads + p.per - 1) / p.per);
  if (units >= 1LL << 30) return fail(MV_ERR_LIMIT, "talk_prefill: %lld tokens", static_cast<long long>(tokens));
  talk_prefill_kernel<NQ><<<static_cast<unsigned>(std::min<int64_t>(units, kNumSMs)), kTpThreads, smem, st>>>(tm[0], tm[1], tm[2], p);
  return check_launch("talk_prefill");
}

}  // namespace mv

extern "C" int mv_talk_prefill_takes(int dim, int vdim, float cap) {
  return dim > 0 && vdim > 0 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 128 && vdim <= 256 && cap > 0.f && cap <= mv::kTalkCap;
}

extern "C" int mv_talk_prefill(void* a, const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v,
                               int64_t v_stride, const int32_t* cu_q, const int32_t* cu_k, int num_seqs, int64_t tokens,
                               int64_t keys, const float* r1, const float* r2, float cap, int heads, int kv_heads, int dim,
                               int vdim, float scale, int* error_word, void* stream) {
  using namespace mv;
  const char* w = "talk_prefill";
  if (num_seqs < 0 || tokens < 0 || keys < tokens || heads <= 0 || kv_heads <= 0 || heads % kv_heads)
    return fail(MV_ERR_SHAPE, "talk_prefill: heads %d over %d, %lld tokens", heads, kv_heads, static_cast<long long>(tokens));
  if (!mv_talk_prefill_takes(dim, vdim, cap)) return fail(MV_ERR_LIMIT, "talk_prefill: dim %d, vdim %d, cap %f", dim, vdim, cap);
  if (tokens == 0 || num_seqs == 0) return MV_OK;
  if (!a || !q || !k || !v || !cu_q || !cu_k || !r1 || !r2 || !error_word) return fail(MV_ERR_NULL, "talk_prefill: null pointer");
  if ((reinterpret_cast<uintptr_t>(a) & 31u) || !vec8_ok(q, q_stride, 2) || !vec8_ok(k, k_stride, 2) || !vec8_ok(v, v_stride, 2))
    return fail(MV_ERR_ALIGN, "talk_prefill: rows must start on 16-byte boundaries");
  CUtensorMap tm[3];
  int rc = make_tmap_bf16(&tm[0], q, dim, heads, tokens, dim, q_stride, 1, kTpTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[1], k, dim, kv_heads, keys, dim, k_stride, 1, kTpTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[2], v, vdim, kv_heads, keys, vdim, v_stride, 1, kTpTile, w);
  if (rc) return rc;
  const int boxes = (vdim + 63) / 64, per = std::min(4 / boxes, kv_heads);
  const TalkPrefillParams p{static_cast<__nv_bfloat16*>(a), cu_q, cu_k, num_seqs, heads, kv_heads, vdim, boxes, per, r1, r2, scale, cap, error_word};
  auto st = static_cast<cudaStream_t>(stream);
  return dim <= 64 ? launch_talk_prefill<1>(tm, p, tokens, st) : launch_talk_prefill<2>(tm, p, tokens, st);
}
