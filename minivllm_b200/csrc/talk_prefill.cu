// Prefill of talking-heads attention (talk_attention.cu) on the Blackwell tensor cores, causal, packed batch.  The mixture of the
// heads' weights is linear, so that it can be taken after the weights have met the values: a CTA forms the weights of ONE head for
// 128 queries and applies them to the values of several value heads, up to 256 columns; head_mix_kernel combines the results.
//
// Scores are capped, so weights are formed against a fixed reference (TalkScore): no running maximum, no rescaling, and the two
// softmax warpgroups take turns at the key tiles of the same queries.
//   warps 0-3 / 4-7  weights of the even / odd key tiles (thread = row = TMEM lane); the bias of a tile's 255 distances, with
//                    -inf behind the query, is put into shared memory while the tile's product is awaited
//   warp 8           TMA producer, warp 9 MMA issuer (S = Q K^T into two buffers, O += P V with P in TMEM)
// Tensor memory: S and P in columns 0-127 and 128-255, O in 256-511.
//
// Per weight: three special functions (two for the cap), or two with the outer power of two on the FMA pipe, against
// 2 (dim + columns) tensor FLOPs: bound by the special-function unit.
#include <algorithm>
#include "mma.cuh"
#include "query_tile.cuh"
#include "talk.cuh"
#include "tcgen05.cuh"
#include "tmap.cuh"
#include "vec.cuh"

namespace mv {

constexpr int kTpThreads = 384, kTpTile = 128;
constexpr int kTpBox = kTpTile * 128;                 // one 64-column box of a 128-row tile
constexpr int kTpTable = 2 * kTpTile;                 // distances of a tile

struct TalkPrefillParams {
  __nv_bfloat16* out;                                 // (tokens, heads, kv_heads, vdim)
  const int32_t *cu_q, *cu_k;
  int num_seqs, heads, kv_heads, vdim;
  int boxes, per;                                     // 64-column boxes of a value head; value heads per CTA
  const float *r1, *r2;
  float scale, cap;
  int* error_word;
};

enum { TB_Q = 0, TB_KFULL = 1, TB_KEMPTY = 3, TB_VFULL = 5, TB_VEMPTY = 7, TB_SFULL = 9, TB_PREADY = 11, TB_ODONE = 13, TB_DRAIN = 14,
       TB_COUNT = 15 };

inline int talk_prefill_kstages(int nq, int boxes) { return nq == 2 && boxes > 3 ? 1 : 2; }
inline int talk_prefill_smem(int nq, int boxes) {
  return ((1 + talk_prefill_kstages(nq, boxes)) * nq + 2 * boxes) * kTpBox + (4 * kTpTable + 2 * kTpTile) * 4 + 1024;
}

__device__ __forceinline__ void group_barrier(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

template <int NQ>
__global__ void __launch_bounds__(kTpThreads, 1)
talk_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                    const __grid_constant__ CUtensorMap tm_v, const TalkPrefillParams p) {
  constexpr int kQBytes = NQ * kTpBox;
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t bars[TB_COUNT];
  __shared__ uint32_t s_tmem;
  __shared__ int s_tile[2], s_scan[kTpThreads / 32], s_abort, s_sticky;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int all = p.per * p.boxes, KS = NQ == 2 && all > 3 ? 1 : 2;
  const uint32_t q_smem = (smem_u32(smem_raw) + 1023u) & ~1023u;      // [box][128][128B]
  const uint32_t k_smem = q_smem + kQBytes;                           // [stage KS][box]
  const uint32_t v_smem = k_smem + KS * kQBytes;                      // [stage 2][box]
  float* s_bias = reinterpret_cast<float*>(smem_raw + (v_smem + 2 * all * kTpBox - smem_u32(smem_raw)));   // [group][buffer][distance]
  float* s_sum = s_bias + 4 * kTpTable;                               // [group][row]
  const uint32_t bar0 = smem_u32(bars);
  auto bar = [&](int i) { return bar0 + 8u * i; };
  volatile int* abort_flag = &s_abort;
  if (tid == 0) {
    s_abort = 0;
    s_sticky = *reinterpret_cast<volatile int*>(p.error_word);
  }
  find_query_tile<kTpThreads>(p.cu_q, p.num_seqs, kTpTile, s_tile, s_scan);
  const int seq = s_tile[0];
  if (seq < 0 || s_sticky != 0) return;      // uniform: the grid is an upper bound; an earlier wait ran out
  const int chunks = (p.kv_heads + p.per - 1) / p.per, head = blockIdx.y / chunks, v0 = (blockIdx.y - head * chunks) * p.per;
  const int kv_head = head / (p.heads / p.kv_heads), v_heads = min(p.per, p.kv_heads - v0), boxes = v_heads * p.boxes;
  const int q_start = p.cu_q[seq], q_len = p.cu_q[seq + 1] - q_start;
  const int k_start = p.cu_k[seq], k_len = p.cu_k[seq + 1] - k_start;
  const int q0 = s_tile[1] * kTpTile, first_pos = k_len - q_len + q0;
  const int n = (k_len - q_len + min(q0 + kTpTile, q_len) + kTpTile - 1) / kTpTile;      // key tiles up to the last row's position

  if (tid == 0) {
    tc::mbar_init(bar(TB_Q), 1);
    for (int s = 0; s < 2; ++s) {
      tc::mbar_init(bar(TB_KFULL + s), 1);
      tc::mbar_init(bar(TB_KEMPTY + s), 1);
      tc::mbar_init(bar(TB_VFULL + s), 1);
      tc::mbar_init(bar(TB_VEMPTY + s), 1);
      tc::mbar_init(bar(TB_SFULL + s), 1);
      tc::mbar_init(bar(TB_PREADY + s), 128);
    }
    tc::mbar_init(bar(TB_ODONE), 1);
    tc::mbar_init(bar(TB_DRAIN), 1);
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
        tc::mbar_expect_tx(bar(TB_Q), kQBytes);
        for (int b = 0; b < NQ; ++b) tc::tma_load_3d(q_smem + b * kTpBox, &tm_q, 64 * b, head, q_start + q0, bar(TB_Q));
        for (int i = 0; i < n; ++i) {
          const int s = i % KS, vs = i & 1, row = k_start + i * kTpTile;
          tc::mbar_wait(bar(TB_KEMPTY + s), ((i / KS) & 1) ^ 1, abort_flag, p.error_word, 1);
          tc::mbar_expect_tx(bar(TB_KFULL + s), kQBytes);
          for (int b = 0; b < NQ; ++b) tc::tma_load_3d(k_smem + s * kQBytes + b * kTpBox, &tm_k, 64 * b, kv_head, row, bar(TB_KFULL + s));
          tc::mbar_wait(bar(TB_VEMPTY + vs), ((i >> 1) & 1) ^ 1, abort_flag, p.error_word, 2);
          tc::mbar_expect_tx(bar(TB_VFULL + vs), boxes * kTpBox);
          for (int b = 0; b < boxes; ++b)
            tc::tma_load_3d(v_smem + (vs * all + b) * kTpBox, &tm_v, 64 * (b % p.boxes), v0 + b / p.boxes, row, bar(TB_VFULL + vs));
        }
        if (*abort_flag) {       // copies in flight must land before the shared memory goes away
          tc::mbar_wait_timed(bar(TB_Q), 0);
          for (int i = max(n - 2, 0); i < n; ++i) {
            if (i >= n - KS) tc::mbar_wait_timed(bar(TB_KFULL + i % KS), (i / KS) & 1);
            tc::mbar_wait_timed(bar(TB_VFULL + (i & 1)), (i >> 1) & 1);
          }
        }
      }
    } else if (warp == 9) {
      const uint32_t idesc_qk = tc::instr_desc_f16(1, 1, false, 128, 128);
      const uint32_t idesc_pv = tc::instr_desc_f16(1, 1, true, 128, 64 * boxes);
      const uint32_t q_lo = tc::desc_lo(q_smem, 16), k_lo = tc::desc_lo(k_smem, 16), v_lo = tc::desc_lo(v_smem, kTpBox);
      auto scores = [&](int i) {           // of tile i, into its buffer
        const int s = i % KS;
        tc::mbar_wait(bar(TB_KFULL + s), (i / KS) & 1, abort_flag, p.error_word, 4);
        tc::fence_after_sync();
        __syncwarp();
#pragma unroll
        for (int b = 0; b < NQ; ++b)
          tc::mma_ss_k64(tmem + (i & 1) * 128, tc::desc64(q_lo + ((b * kTpBox) >> 4), tc::kDescHiSw128Sbo1024),
                         tc::desc64(k_lo + ((s * kQBytes + b * kTpBox) >> 4), tc::kDescHiSw128Sbo1024), idesc_qk, b > 0);
        tc::commit_elected(bar(TB_SFULL + (i & 1)), bar(TB_KEMPTY + s), true);
      };
      tc::mbar_wait(bar(TB_Q), 0, abort_flag, p.error_word, 3);
      scores(0);
      if (n > 1) scores(1);
      for (int i = 0; i < n; ++i) {
        const int vs = i & 1;
        tc::mbar_wait(bar(TB_VFULL + vs), (i >> 1) & 1, abort_flag, p.error_word, 5);
        tc::mbar_wait(bar(TB_PREADY + vs), (i >> 1) & 1, abort_flag, p.error_word, 7);
        tc::fence_after_sync();
        __syncwarp();
        tc::mma_ts_k128_commit(tmem + 256, tmem + vs * 128, tc::desc64(v_lo + ((vs * all * kTpBox) >> 4), tc::kDescHiSw128Sbo1024),
                               idesc_pv, i > 0, bar(TB_VEMPTY + vs));
        if (i + 2 < n) scores(i + 2);
      }
      tc::commit_elected(bar(TB_ODONE), 0, false);
      if (*abort_flag) {
        __syncwarp();
        tc::commit_elected(bar(TB_DRAIN), 0, false);
        tc::mbar_wait_timed(bar(TB_DRAIN), 0);
      }
    }
  } else {
    tc::setmaxnreg_inc_232();
    const int t = warp >> 2, row = (warp & 3) * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t s_addr = tmem + lane_addr + t * 128, o_addr = tmem + lane_addr + 256;
    const TalkScore score(p.scale, p.cap);
    const float r1 = p.r1[head], r2 = p.r2[head];
    const float2 in2 = make_float2(score.in, score.in), out2 = make_float2(score.out, score.out), one2 = make_float2(1.f, 1.f);
    float l = 0.f;
    for (int i = t, k = 0; i < n; i += 2, ++k) {
      float* tab = s_bias + (t * 2 + (k & 1)) * kTpTable;
      const int d0 = first_pos - i * kTpTile - (kTpTile - 1);        // distance of the first row to the last key
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int d = d0 + row + x * kTpTile;
        tab[row + x * kTpTile] = d < 0 ? -INFINITY : score.bias(r1, r2, d);
      }
      group_barrier(2 + t, 128);
      tc::mbar_wait(bar(TB_SFULL + t), k & 1, abort_flag, p.error_word, 8);
      tc::fence_after_sync();
      uint32_t sv[4][32];
#pragma unroll
      for (int c = 0; c < 4; ++c) tc::tmem_ld32(s_addr + c * 32, sv[c]);
      tc::wait_ld();
      const float* mine = tab + row + (kTpTile - 1);                 // the bias of key col is mine[-col]
      float2 sums[4] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
      for (int c2 = 0; c2 < 2; ++c2) {
        uint32_t pk[32];
#pragma unroll
        for (int y = 0; y < 32; ++y) {
          const int c = 2 * c2 + (y >> 4), col = (y & 15) * 2;
          const float2 z = mul_f32x2(make_float2(__uint_as_float(sv[c][col]), __uint_as_float(sv[c][col + 1])), in2);
          const float2 d = tc::add2(make_float2(tc::ex2_mufu(z.x), tc::ex2_mufu(z.y)), one2);
          const float2 x = tc::fma2(make_float2(fast_rcp(d.x), fast_rcp(d.y)), out2,
                                    make_float2(mine[-(c * 32 + col)], mine[-(c * 32 + col + 1)]));
          float2 e;
          if ((y & 3) != 3) {
            e = tc::ex2_poly2(x);
          } else {
            e.x = tc::ex2_mufu(x.x);
            e.y = tc::ex2_mufu(x.y);
          }
          sums[y & 3] = tc::add2(sums[y & 3], e);
          pk[y] = pack2<__nv_bfloat16>(e.x, e.y);
        }
        tc::tmem_st32(s_addr + c2 * 32, pk);
      }
      const float2 s01 = tc::add2(sums[0], sums[1]), s23 = tc::add2(sums[2], sums[3]);
      l += (s01.x + s01.y) + (s23.x + s23.y);
      tc::wait_st();
      tc::fence_before_sync();
      tc::mbar_arrive(bar(TB_PREADY + t));
    }
    s_sum[t * kTpTile + row] = l;
    group_barrier(1, 256);
    l = s_sum[row] + s_sum[kTpTile + row];
    const float inv = l > 0.f ? 1.f / l : 0.f;
    tc::mbar_wait(bar(TB_ODONE), 0, abort_flag, p.error_word, 10);
    tc::fence_after_sync();
    const int qrow = q0 + row;
    __nv_bfloat16* orow = p.out + (static_cast<int64_t>(q_start + qrow) * p.heads + head) * p.kv_heads * p.vdim;
#pragma unroll 1
    for (int c = t * boxes; c < (t + 1) * boxes; ++c) {              // 32 columns at a time, half of them per group
      const int vh = c / (2 * p.boxes), d0 = (c - vh * 2 * p.boxes) * 32;
      uint32_t ov[32];
      tc::tmem_ld32(o_addr + c * 32, ov);
      tc::wait_ld();
      if (qrow < q_len) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (d0 + i * 8 >= p.vdim) continue;
          uint4 w;
          w.x = pack2<__nv_bfloat16>(__uint_as_float(ov[8 * i + 0]) * inv, __uint_as_float(ov[8 * i + 1]) * inv);
          w.y = pack2<__nv_bfloat16>(__uint_as_float(ov[8 * i + 2]) * inv, __uint_as_float(ov[8 * i + 3]) * inv);
          w.z = pack2<__nv_bfloat16>(__uint_as_float(ov[8 * i + 4]) * inv, __uint_as_float(ov[8 * i + 5]) * inv);
          w.w = pack2<__nv_bfloat16>(__uint_as_float(ov[8 * i + 6]) * inv, __uint_as_float(ov[8 * i + 7]) * inv);
          st_global16(orow + (v0 + vh) * p.vdim + d0 + i * 8, w);
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

template <int NQ>
static int launch_talk_prefill(const CUtensorMap (&tm)[3], const TalkPrefillParams& p, int64_t tokens, cudaStream_t st) {
  const int smem = talk_prefill_smem(NQ, p.per * p.boxes);
  const cudaError_t e = cudaFuncSetAttribute(talk_prefill_kernel<NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return fail(MV_ERR_CUDA, "talk_prefill: %s", cudaGetErrorString(e));
  const dim3 grid(static_cast<unsigned>(tokens / kTpTile + std::min<int64_t>(p.num_seqs, tokens)), p.heads * ((p.kv_heads + p.per - 1) / p.per));
  talk_prefill_kernel<NQ><<<grid, kTpThreads, smem, st>>>(tm[0], tm[1], tm[2], p);
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
  if (!aligned16(a) || !vec8_ok(q, q_stride, 2) || !vec8_ok(k, k_stride, 2) || !vec8_ok(v, v_stride, 2))
    return fail(MV_ERR_ALIGN, "talk_prefill: rows must start on 16-byte boundaries");
  CUtensorMap tm[3];
  int rc = make_tmap_bf16(&tm[0], q, dim, heads, tokens, dim, q_stride, 1, kTpTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[1], k, dim, kv_heads, keys, dim, k_stride, 1, kTpTile, w);
  if (!rc) rc = make_tmap_bf16(&tm[2], v, vdim, kv_heads, keys, vdim, v_stride, 1, kTpTile, w);
  if (rc) return rc;
  const int boxes = (vdim + 63) / 64, per = std::min(4 / boxes, kv_heads);
  const TalkPrefillParams p{static_cast<__nv_bfloat16*>(a), cu_q, cu_k, num_seqs, heads, kv_heads, vdim, boxes, per, r1, r2, scale, cap, error_word};
  auto st = static_cast<cudaStream_t>(stream);
  if (static_cast<int64_t>(heads) * ((kv_heads + per - 1) / per) > 65535) return fail(MV_ERR_LIMIT, "talk_prefill: heads %d over %d", heads, kv_heads);
  return dim <= 64 ? launch_talk_prefill<1>(tm, p, tokens, st) : launch_talk_prefill<2>(tm, p, tokens, st);
}
