// Mixture of experts: routing, the stable sort of (token, choice) pairs by expert, the gather of the rows, and a
// grouped matrix product for any sizes in bf16 or fp32 (the tensor-core form is in grouped_gemm.cu).
//
// Everything that depends on the routing stays on the device: the products read the experts' row ranges from
// `offsets`, so a step needs no host synchronisation and can be captured in a graph.  A token's result does not
// depend on the batch: rows are computed one by one and combined in the order of the token's own choices.
#include <algorithm>
#include "vec.cuh"

namespace mv {

constexpr int kRtThreads = 256;
constexpr int kRtMaxPer = 32;      // experts per lane: up to 1024 experts

// One warp per token: the `top` largest logits (ties: lower index) and the softmax over them (kAll: over all experts), times
// `scale`.
// kPer: experts per lane.
template <int kPer, bool kAll>
__global__ void __launch_bounds__(kRtThreads)
moe_route_kernel(int32_t* __restrict__ idx, float* __restrict__ weight, const float* __restrict__ logits,
                 int64_t stride, const float* __restrict__ bias, int64_t tokens, int experts, int top, int groups,
                 int keep, float scale) {
  __shared__ float s_best[kRtThreads / 32][32 * kPer];      // per group of experts: its largest logit
  const int lane = threadIdx.x & 31;
  const int64_t t = static_cast<int64_t>(blockIdx.x) * (kRtThreads / 32) + (threadIdx.x >> 5);
  if (t >= tokens) return;
  float z[kPer];
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int e = i * 32 + lane;
    z[i] = e < experts ? logits[t * stride + e] + (bias ? bias[e] : 0.f) : -INFINITY;
  }
  uint32_t taken = 0;
  if (groups > 1) {
    // a group is dropped when `keep` groups come before it (larger maximum, ties: lower index)
    float* best = s_best[threadIdx.x >> 5];
    const int size = experts / groups;
    for (int i = lane; i < groups; i += 32) {
      float m = -INFINITY;
      for (int e = i * size; e < (i + 1) * size; ++e) m = fmaxf(m, logits[t * stride + e] + (bias ? bias[e] : 0.f));
      best[i] = m;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int e = i * 32 + lane;
      if (e < experts) {
        const int mine = e / size;
        const float m = best[mine];
        int before = 0;
        for (int g = 0; g < groups; ++g) before += best[g] > m || (best[g] == m && g < mine);
        if (before >= keep) taken |= 1u << i;
      }
    }
  }
  float first = 0.f, sum = 0.f;
  if (kAll) {
#pragma unroll
    for (int i = 0; i < kPer; ++i) first = i == 0 ? z[0] : fmaxf(first, z[i]);
#pragma unroll
    for (int o = 16; o; o >>= 1) first = fmaxf(first, __shfl_xor_sync(0xffffffffu, first, o));
#pragma unroll
    for (int i = 0; i < kPer; ++i) sum += i * 32 + lane < experts ? expf(z[i] - first) : 0.f;
    sum = warp_sum(sum);
  }
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int e = i * 32 + lane;
      if (e < experts && !((taken >> i) & 1u) && (z[i] > best || at == 0x7fffffff)) { best = z[i]; at = e; }
    }
#pragma unroll
    for (int o = 16; o; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (oa != 0x7fffffff && (at == 0x7fffffff || ob > best || (ob == best && oa < at))) { best = ob; at = oa; }
    }
    if ((at & 31) == lane) taken |= 1u << (at >> 5);
    if (!kAll && k == 0) first = best;
    const float e = expf(best - first);
    if (!kAll) sum += e;
    if (lane == 0) {
      idx[t * top + k] = at;
      weight[t * top + k] = e;
    }
  }
  __syncwarp();
  for (int k = lane; k < top; k += 32) weight[t * top + k] = weight[t * top + k] / sum * scale;
}

constexpr int kSortThreads = 256;   // entries per block

__global__ void __launch_bounds__(kSortThreads)
moe_count_kernel(int32_t* __restrict__ hist, const int32_t* __restrict__ idx, int64_t entries, int experts) {
  extern __shared__ int s_h[];
  for (int e = threadIdx.x; e < experts; e += kSortThreads) s_h[e] = 0;
  __syncthreads();
  const int64_t i = static_cast<int64_t>(blockIdx.x) * kSortThreads + threadIdx.x;
  if (i < entries) atomicAdd(&s_h[idx[i]], 1);
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += kSortThreads) hist[static_cast<int64_t>(blockIdx.x) * experts + e] = s_h[e];
}

// One CTA: hist[b][e] becomes the first row of block b's entries of expert e; offsets[e] the expert's first row.
// The 1,024 threads are `ep` experts (a power of two) times 1,024 / ep runs of blocks.
__global__ void __launch_bounds__(1024)
moe_scan_kernel(int32_t* __restrict__ hist, int32_t* __restrict__ offsets, int blocks, int experts, int ep) {
  __shared__ int s_run[1024], s_tot[1024];
  const int tid = threadIdx.x, e = tid & (ep - 1), seg = tid / ep, segs = 1024 / ep;
  const int per = (blocks + segs - 1) / segs, b0 = min(seg * per, blocks), b1 = min(b0 + per, blocks);
  int sum = 0;
  if (e < experts) {
#pragma unroll 8
    for (int b = b0; b < b1; ++b) sum += hist[static_cast<int64_t>(b) * experts + e];
  }
  s_run[tid] = sum;
  s_tot[tid] = 0;
  __syncthreads();
  if (seg == 0) {
    int total = 0;
    for (int k = 0; k < segs; ++k) {
      const int v = s_run[k * ep + e];
      s_run[k * ep + e] = total;       // entries of the runs before
      total += v;
    }
    s_tot[e] = total;
  }
  __syncthreads();
  const int mine = s_tot[tid];
  for (int o = 1; o < ep; o <<= 1) {
    const int v = tid >= o ? s_tot[tid - o] : 0;
    __syncthreads();
    s_tot[tid] += v;
    __syncthreads();
  }
  if (tid < experts) offsets[tid] = s_tot[tid] - mine;
  if (tid == experts - 1) offsets[experts] = s_tot[tid];
  if (e >= experts) return;
  int run = (e ? s_tot[e - 1] : 0) + s_run[tid];
#pragma unroll 4
  for (int b = b0; b < b1; ++b) {
    const int64_t a = static_cast<int64_t>(b) * experts + e;
    const int n = hist[a];
    hist[a] = run;
    run += n;
  }
}

// pos[entry] = sorted row of the entry; row_token[row] = its token.
__global__ void __launch_bounds__(kSortThreads)
moe_place_kernel(int32_t* __restrict__ pos, int32_t* __restrict__ row_token, const int32_t* __restrict__ base,
                 const int32_t* __restrict__ idx, int64_t entries, int experts, int top) {
  __shared__ int s_e[kSortThreads];
  const int64_t i = static_cast<int64_t>(blockIdx.x) * kSortThreads + threadIdx.x;
  const int e = i < entries ? idx[i] : -1;
  s_e[threadIdx.x] = e;
  __syncthreads();
  if (e < 0) return;
  int rank = 0;
  for (int j = 0; j < threadIdx.x; ++j) rank += s_e[j] == e;
  const int row = base[static_cast<int64_t>(blockIdx.x) * experts + e] + rank;
  pos[i] = row;
  row_token[row] = static_cast<int32_t>(i / top);
}

// The three steps above in one CTA, for the few entries of a decode step.
constexpr int kSmallEntries = 2048;
__global__ void __launch_bounds__(1024)
moe_sort_small_kernel(int32_t* __restrict__ pos, int32_t* __restrict__ row_token, int32_t* __restrict__ offsets,
                      const int32_t* __restrict__ idx, int entries, int experts, int top) {
  __shared__ int s_e[kSmallEntries];
  __shared__ int s_tot[1024];
  const int tid = threadIdx.x;
  s_tot[tid] = 0;
  __syncthreads();
  for (int i = tid; i < entries; i += 1024) {
    s_e[i] = idx[i];
    atomicAdd(&s_tot[s_e[i]], 1);
  }
  __syncthreads();
  const int mine = s_tot[tid];
  for (int o = 1; o < 1024; o <<= 1) {
    const int v = tid >= o ? s_tot[tid - o] : 0;
    __syncthreads();
    s_tot[tid] += v;
    __syncthreads();
  }
  const int first = s_tot[tid] - mine;
  __syncthreads();
  s_tot[tid] = first;
  if (tid < experts) offsets[tid] = first;
  if (tid == experts - 1) offsets[experts] = first + mine;
  __syncthreads();
  for (int i = tid; i < entries; i += 1024) {
    const int e = s_e[i];
    int rank = 0;
    for (int j = 0; j < i; ++j) rank += s_e[j] == e;
    const int row = s_tot[e] + rank;
    pos[i] = row;
    row_token[row] = i / top;
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
gather_rows_kernel(T* __restrict__ out, const T* __restrict__ x, int64_t x_stride, const int32_t* __restrict__ row_token,
                   int64_t rows, int width) {
  const int per = width / V;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < rows * per; i += static_cast<int64_t>(gridDim.x) * 256) {
    const int64_t r = i / per;
    const int c = static_cast<int>(i - r * per) * V;
    if (V == 8 && sizeof(T) == 2) {
      *reinterpret_cast<uint4*>(out + r * width + c) = *reinterpret_cast<const uint4*>(x + row_token[r] * x_stride + c);
    } else {
      float v[V];
      Vec<T, V>::load(x + row_token[r] * x_stride + c, v);
      Vec<T, V>::store(out + r * width + c, v);
    }
  }
}

// Grouped product, plain form: rows [offsets[e], offsets[e+1]) of x times w[e] (out_dim, in_dim) transposed.
// kGated: w[e] holds 2 * out_dim rows (gate, then up) and the result is the gate applied to up (glu_act).
constexpr int kGgRows = 32, kGgCols = 64, kGgK = 32, kGgThreads = 256;
template <typename T, bool kGated>
__global__ void __launch_bounds__(kGgThreads)
grouped_rows_kernel(T* __restrict__ out, const T* __restrict__ x, const T* __restrict__ w,
                    const int32_t* __restrict__ offsets, int experts, int in_dim, int out_dim, int act, float limit) {
  __shared__ float sx[kGgRows][kGgK + 1], sw[kGated ? 2 : 1][kGgCols][kGgK + 1];
  __shared__ int s_e, s_r0, s_r1;
  if (threadIdx.x == 0) {
    int tile = blockIdx.y, e = 0;
    s_e = -1;
    for (; e < experts; ++e) {
      const int n = offsets[e + 1] - offsets[e], tiles = (n + kGgRows - 1) / kGgRows;
      if (tile < tiles) {
        s_e = e;
        s_r0 = offsets[e] + tile * kGgRows;
        s_r1 = min(s_r0 + kGgRows, offsets[e + 1]);
        break;
      }
      tile -= tiles;
    }
  }
  __syncthreads();
  if (s_e < 0) return;
  const int r0 = s_r0, nr = s_r1 - s_r0, c0 = blockIdx.x * kGgCols;
  const T* we = w + static_cast<int64_t>(s_e) * (kGated ? 2 : 1) * out_dim * in_dim;
  const int tr = threadIdx.x / 16, tc = threadIdx.x % 16;   // 2 rows x 4 columns per thread
  float acc[kGated ? 2 : 1][2][4] = {};
  for (int k0 = 0; k0 < in_dim; k0 += kGgK) {
    for (int i = threadIdx.x; i < kGgRows * kGgK; i += kGgThreads) {
      const int r = i / kGgK, k = k0 + i % kGgK;
      sx[r][i % kGgK] = r < nr && k < in_dim ? Elem<T>::to_f(x[static_cast<int64_t>(r0 + r) * in_dim + k]) : 0.f;
    }
    for (int i = threadIdx.x; i < kGgCols * kGgK; i += kGgThreads) {
      const int c = i / kGgK, k = k0 + i % kGgK;
#pragma unroll
      for (int m = 0; m < (kGated ? 2 : 1); ++m)
        sw[m][c][i % kGgK] = c0 + c < out_dim && k < in_dim
            ? Elem<T>::to_f(we[(static_cast<int64_t>(m) * out_dim + c0 + c) * in_dim + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < kGgK; ++k) {
      const float a0 = sx[tr * 2][k], a1 = sx[tr * 2 + 1][k];
#pragma unroll
      for (int m = 0; m < (kGated ? 2 : 1); ++m)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float b = sw[m][tc + 16 * j][k];
          acc[m][0][j] = fmaf(a0, b, acc[m][0][j]);
          acc[m][1][j] = fmaf(a1, b, acc[m][1][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = tr * 2 + i;
    if (r >= nr) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = c0 + tc + 16 * j;
      if (c >= out_dim) continue;
      const float v = kGated ? glu_act<float>(act, acc[0][i][j], acc[kGated ? 1 : 0][i][j], limit) : acc[0][i][j];
      out[static_cast<int64_t>(r0 + r) * out_dim + c] = Elem<T>::from_f(v);
    }
  }
}

}  // namespace mv

extern "C" int mv_moe_route(int32_t* idx, float* weight, const float* logits, int64_t logits_stride, const float* bias,
                            int64_t tokens, int experts, int top, int groups, int keep, int over_all, float scale, void* stream) {
  using namespace mv;
  if (tokens < 0 || experts <= 0 || top <= 0 || top > experts) return fail(MV_ERR_SHAPE, "moe_route: experts %d top %d", experts, top);
  if (groups <= 0 || experts % groups || keep <= 0 || keep > groups || experts / groups * keep < top)
    return fail(MV_ERR_SHAPE, "moe_route: %d groups of %d experts, %d kept, top %d", groups, experts, keep, top);
  if (experts > 32 * kRtMaxPer) return fail(MV_ERR_LIMIT, "moe_route: %d experts (at most %d)", experts, 32 * kRtMaxPer);
  if (tokens == 0) return MV_OK;
  if (!idx || !weight || !logits) return fail(MV_ERR_NULL, "moe_route: null pointer");
  const unsigned grid = static_cast<unsigned>((tokens + kRtThreads / 32 - 1) / (kRtThreads / 32));
  auto go = [&](auto kernel) {
    kernel<<<grid, kRtThreads, 0, static_cast<cudaStream_t>(stream)>>>(idx, weight, logits, logits_stride, bias, tokens, experts, top,
                                                                        keep < groups ? groups : 1, keep, scale);
  };
  if (experts <= 64) over_all ? go(moe_route_kernel<2, true>) : go(moe_route_kernel<2, false>);
  else if (experts <= 256) over_all ? go(moe_route_kernel<8, true>) : go(moe_route_kernel<8, false>);
  else over_all ? go(moe_route_kernel<kRtMaxPer, true>) : go(moe_route_kernel<kRtMaxPer, false>);
  return check_launch("moe_route");
}

extern "C" int64_t mv_moe_sort_workspace_bytes(int64_t tokens, int experts, int top) {
  using namespace mv;
  const int64_t entries = tokens * top;
  if (entries <= kSmallEntries) return 0;
  return (entries + kSortThreads - 1) / kSortThreads * experts * 4;
}

extern "C" int mv_moe_sort(int32_t* pos, int32_t* row_token, int32_t* offsets, const int32_t* idx, int64_t tokens,
                           int experts, int top, void* workspace, int64_t workspace_bytes, void* stream) {
  using namespace mv;
  if (tokens < 0 || experts <= 0 || top <= 0) return fail(MV_ERR_SHAPE, "moe_sort: experts %d top %d", experts, top);
  if (experts > 1024) return fail(MV_ERR_LIMIT, "moe_sort: %d experts (at most 1024)", experts);
  if (!offsets || (tokens && (!pos || !row_token || !idx))) return fail(MV_ERR_NULL, "moe_sort: null pointer");
  auto st = static_cast<cudaStream_t>(stream);
  const int64_t entries = tokens * top;
  if (entries <= kSmallEntries) {
    moe_sort_small_kernel<<<1, 1024, 0, st>>>(pos, row_token, offsets, idx, static_cast<int>(entries), experts, top);
    return check_launch("moe_sort");
  }
  const int blocks = static_cast<int>((entries + kSortThreads - 1) / kSortThreads);
  if (!workspace || workspace_bytes < static_cast<int64_t>(blocks) * experts * 4) return fail(MV_ERR_WORKSPACE, "moe_sort: workspace");
  auto* hist = static_cast<int32_t*>(workspace);
  moe_count_kernel<<<blocks, kSortThreads, experts * sizeof(int), st>>>(hist, idx, entries, experts);
  int ep = 1;
  while (ep < experts) ep *= 2;
  moe_scan_kernel<<<1, 1024, 0, st>>>(hist, offsets, blocks, experts, ep);
  moe_place_kernel<<<blocks, kSortThreads, 0, st>>>(pos, row_token, hist, idx, entries, experts, top);
  return check_launch("moe_sort");
}

extern "C" int mv_gather_rows(void* out, const void* x, int64_t x_stride, const int32_t* row_token, int64_t rows,
                              int width, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "gather_rows: dtype %d", dtype);
  if (rows < 0 || width <= 0) return fail(MV_ERR_SHAPE, "gather_rows: width %d", width);
  if (rows == 0) return MV_OK;
  if (!out || !x || !row_token) return fail(MV_ERR_NULL, "gather_rows: null pointer");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int eb = sizeof(T);
    const bool v8 = width % 8 == 0 && aligned16(out) && vec8_ok(x, x_stride, eb);
    const int64_t work = rows * (v8 ? width / 8 : width);
    const unsigned grid = static_cast<unsigned>(std::min<int64_t>((work + 255) / 256, kNumSMs * 16));
    auto st = static_cast<cudaStream_t>(stream);
    if (v8) gather_rows_kernel<T, 8><<<grid, 256, 0, st>>>(static_cast<T*>(out), static_cast<const T*>(x), x_stride, row_token, rows, width);
    else gather_rows_kernel<T, 1><<<grid, 256, 0, st>>>(static_cast<T*>(out), static_cast<const T*>(x), x_stride, row_token, rows, width);
    return check_launch("gather_rows");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_grouped_rows(void* out, const void* x, const void* w, const int32_t* offsets, int experts,
                               int64_t rows, int in_dim, int out_dim, int act, float limit, int dtype, void* stream) {
  using namespace mv;
  if (act < MV_ACT_NONE || act > MV_ACT_RELU) return fail(MV_ERR_SHAPE, "grouped_rows: activation %d", act);
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "grouped_rows: dtype %d", dtype);
  if (rows < 0 || experts <= 0 || in_dim <= 0 || out_dim <= 0) return fail(MV_ERR_SHAPE, "grouped_rows: %d x %d", out_dim, in_dim);
  if (rows == 0) return MV_OK;
  if (!out || !x || !w || !offsets) return fail(MV_ERR_NULL, "grouped_rows: null pointer");
  // every expert has at most one partly filled tile
  const int64_t tiles = rows / kGgRows + std::min<int64_t>(experts, rows);
  if (tiles > 65535) return fail(MV_ERR_LIMIT, "grouped_rows: %lld rows", static_cast<long long>(rows));
  const dim3 grid((out_dim + kGgCols - 1) / kGgCols, static_cast<unsigned>(tiles));
  auto st = static_cast<cudaStream_t>(stream);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto* o = static_cast<T*>(out);
    auto *a = static_cast<const T*>(x), *b = static_cast<const T*>(w);
    if (act != MV_ACT_NONE) grouped_rows_kernel<T, true><<<grid, kGgThreads, 0, st>>>(o, a, b, offsets, experts, in_dim, out_dim, act, limit);
    else grouped_rows_kernel<T, false><<<grid, kGgThreads, 0, st>>>(o, a, b, offsets, experts, in_dim, out_dim, act, limit);
    return check_launch("grouped_rows");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}
