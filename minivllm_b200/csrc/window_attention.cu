// Grouped-query attention with a sliding window, a learned bias per distance and head, and a sink per head, over a paged
// cache of rows [keys of all KV heads | values of all KV heads] (key and value sizes may differ).  Position i sees the
// keys j with 0 <= i - j < window; score = scale (q . k) + bias[h][min(i - j, distances - 1)]; exp(sink[h]) joins the
// denominator.  Bias and sink may be absent.  With a rotation table the result of position i is turned by -i in pairs of
// neighbouring columns (values that were turned by their own positions when they were stored).
//
// kv_norm_store_kernel        RMS norm over all query rows and over all key rows of a token, scatter of [k | v]
// Two more forms of attention over the same kind of cache run on the kernel for any sizes (and on kernels of their own,
// talk_attention.cu, diff_attention.cu):
//   capped scores, a bias that grows with the logarithm of the distance, every weight head's result for every value head;
//   keys in `maps` heads per value head, positions that see their own chunk of the sequence only.
//
// qkv_rope_store_kernel       RMS norm and rotation per query and key head, rotation of the values, scatter of [k | v]
// window_attention_rows_kernel  any sizes, bf16 or fp32, token by token
// window_decode_kernel        one token per sequence on mma.sync: HBM-bound on the rows inside the window
// Portions of prompts run on tcgen05 in latent_prefill.cu.
#include <algorithm>
#include <type_traits>
#include "mma.cuh"
#include "vec.cuh"

namespace mv {

constexpr int kKnThreads = 256;

template <typename T, int V>
__global__ void __launch_bounds__(kKnThreads)
kv_norm_store_kernel(T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int64_t stride,
                     const T* __restrict__ q_weight, const T* __restrict__ k_weight, T* __restrict__ kv_out,
                     T* __restrict__ cache, const int64_t* __restrict__ slot_mapping, int64_t num_slots, int qn, int kn,
                     int vn, float eps) {
  __shared__ float part[2][kKnThreads / 32];
  const int64_t t = blockIdx.x;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  T* qr = q + t * stride;
  const T *kr = k + t * stride, *vr = v + t * stride;
  const int row = kn + vn;
  T* lo = kv_out ? kv_out + t * row : nullptr;
  T* co = nullptr;
  if (cache) {
    const int64_t slot = slot_mapping[t];
    if (slot >= 0 && slot < num_slots) co = cache + slot * row;
  }
  // the first pieces stay in registers: rows of up to 2,048 queries and keys are read once
  constexpr int kHold = 2;
  float hold[kHold][V];
  float a = 0.f, b = 0.f;
  for (int i = tid, n = 0; i < (qn + kn) / V; i += kKnThreads, ++n) {
    const int c = i * V;
    float x[V];
    Vec<T, V>::load(c < qn ? qr + c : kr + c - qn, x);
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < V; ++e) s = fmaf(x[e], x[e], s);
    if (c < qn) a += s; else b += s;
#pragma unroll
    for (int h = 0; h < kHold; ++h)
      if (h == n)
#pragma unroll
        for (int e = 0; e < V; ++e) hold[h][e] = x[e];
  }
  a = warp_sum(a);
  b = warp_sum(b);
  if (lane == 0) { part[0][warp] = a; part[1][warp] = b; }
  for (int i = tid; i < vn / V; i += kKnThreads) {
    float x[V];
    Vec<T, V>::load(vr + i * V, x);
    if (lo) Vec<T, V>::store(lo + kn + i * V, x);
    if (co) Vec<T, V>::store(co + kn + i * V, x);
  }
  __syncthreads();
  a = b = 0.f;
  for (int w = 0; w < kKnThreads / 32; ++w) { a += part[0][w]; b += part[1][w]; }
  const float rq = 1.f / sqrtf(a / static_cast<float>(qn) + eps), rk = 1.f / sqrtf(b / static_cast<float>(kn) + eps);
  for (int i = tid, n = 0; i < (qn + kn) / V; i += kKnThreads, ++n) {
    const int c = i * V;
    const bool is_q = c < qn;
    float x[V], w[V];
    if (n >= kHold) Vec<T, V>::load(is_q ? qr + c : kr + c - qn, x);
#pragma unroll
    for (int h = 0; h < kHold; ++h)
      if (h == n)
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = hold[h][e];
    Vec<T, V>::load(is_q ? q_weight + c : k_weight + c - qn, w);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = x[e] * (is_q ? rq : rk) * w[e];
    if (is_q) {
      Vec<T, V>::store(qr + c, x);
    } else {
      if (lo) Vec<T, V>::store(lo + c - qn, x);
      if (co) Vec<T, V>::store(co + c - qn, x);
    }
  }
}

// Row of a rotation table; padding rows have positions below zero.
__device__ __forceinline__ int64_t table_row(int64_t pos, int64_t rows) { return min(max(pos, static_cast<int64_t>(0)), rows - 1); }

// The pairs of neighbouring columns c .. c + V - 1 of a row of `dims` rotated columns, turned by the table's angles.
template <int V>
__device__ __forceinline__ void turn_pairs(float (&x)[V], int c, int dims, const float* __restrict__ cos_row, const float* __restrict__ sin_row) {
  if (V == 8 && dims % 8 == 0) {         // rows of whole 16-byte pieces
    if (c >= dims) return;
    const float4 co = __ldg(reinterpret_cast<const float4*>(cos_row + c / 2)), si = __ldg(reinterpret_cast<const float4*>(sin_row + c / 2));
    const float cs[4] = {co.x, co.y, co.z, co.w}, sn[4] = {si.x, si.y, si.z, si.w};
#pragma unroll
    for (int e = 0; e < V / 2; ++e) {
      const float a = x[2 * e], b = x[2 * e + 1];
      x[2 * e] = a * cs[e & 3] - b * sn[e & 3];
      x[2 * e + 1] = b * cs[e & 3] + a * sn[e & 3];
    }
    return;
  }
#pragma unroll
  for (int e = 0; e < V; e += 2) {
    if (c + e >= dims) return;
    const float co = cos_row[(c + e) / 2], si = sin_row[(c + e) / 2], a = x[e], b = x[e + 1];
    x[e] = a * co - b * si;
    x[e + 1] = b * co + a * si;
  }
}
// A pair turned by the opposite of an angle, given as (cos, sin).
__device__ __forceinline__ void turn_back(float& a, float& b, float2 cs) {
  const float x = fmaf(a, cs.x, b * cs.y);
  b = fmaf(b, cs.x, -a * cs.y);
  a = x;
}

template <typename T> struct RopeStoreParams {
  T *q; const T *k, *v; int64_t stride;        // (tokens, heads * dim), (tokens, kv_heads * dim), (tokens, kv_heads * vdim)
  const T *q_weight, *k_weight, *temp;         // (dim), (dim; null: keys are stored as they are), (heads) or null
  const float *cos_t, *sin_t; int dims;        // (table_rows, dims / 2)
  const float *vcos_t, *vsin_t;                // (table_rows, vdim / 2), null: values are stored as they are
  int64_t table_rows;
  const int64_t* positions;
  T *kv_out, *cache; const int64_t* slot_mapping; int64_t num_slots;
  int64_t tokens;
  int heads, kv_heads, v_heads, dim, vdim;
  float eps;
};

// L lanes (a power of two) per head of a token, kCh pieces of V (8, or 2 for any sizes) columns per lane.  Items of a token: query heads, key heads,
// value heads.
template <typename T, int V, int L, int kCh>
__global__ void __launch_bounds__(kKnThreads) qkv_rope_store_kernel(const RopeStoreParams<T> p) {
  const int lane = threadIdx.x & (L - 1), per = p.heads + p.kv_heads + p.v_heads, row = p.kv_heads * p.dim + p.v_heads * p.vdim;
  const uint32_t items = static_cast<uint32_t>(p.tokens * per), step = gridDim.x * (kKnThreads / L);      // the host checks the range
  for (uint32_t i0 = blockIdx.x * (kKnThreads / L); i0 < items; i0 += step) {
    const uint32_t i = i0 + threadIdx.x / L, row_i = i / static_cast<uint32_t>(per);
    const bool on = i < items;                 // lanes of a warp stay together for the sums
    const int64_t t = on ? row_i : 0;
    const int item = on ? static_cast<int>(i - row_i * per) : 0;
    const bool is_q = item < p.heads, is_v = item >= p.heads + p.kv_heads;
    const int head = is_q ? item : is_v ? item - p.heads - p.kv_heads : item - p.heads, n = is_v ? p.vdim : p.dim;
    const T* src = is_q ? p.q : is_v ? p.v : p.k;
    src += t * p.stride + static_cast<int64_t>(head) * n;
    const int64_t pos = table_row(p.positions[t], p.table_rows);
    float x[kCh][V], acc = 0.f;
#pragma unroll
    for (int k = 0; k < kCh; ++k) {
      const int c = (k * L + lane) * V;
      if (on && c < n) {
        if constexpr (V == 8) {
          Vec<T, V>::load(src + c, x[k]);
        } else {
          x[k][0] = Elem<T>::to_f(src[c]);
          x[k][1] = c + 1 < n ? Elem<T>::to_f(src[c + 1]) : 0.f;
        }
#pragma unroll
        for (int e = 0; e < V; ++e) acc = fmaf(x[k][e], x[k][e], acc);
      }
    }
#pragma unroll
    for (int o = L / 2; o; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    const T* weight = is_q ? p.q_weight : p.k_weight;
    const float rs = 1.f / sqrtf(acc / static_cast<float>(n) + p.eps);
    const float f = is_q && p.temp && on ? Elem<T>::to_f(p.temp[head]) : 1.f;
    const float* co = is_v ? p.vcos_t : p.cos_t;
    const float* si = is_v ? p.vsin_t : p.sin_t;
    const int dims = is_v ? (co ? p.vdim : 0) : p.dims;
    T *d0 = nullptr, *d1 = nullptr;
    if (is_q) {
      d0 = p.q + t * p.stride + static_cast<int64_t>(head) * n;
    } else {
      const int64_t at = is_v ? static_cast<int64_t>(p.kv_heads) * p.dim + static_cast<int64_t>(head) * n : static_cast<int64_t>(head) * n;
      if (p.kv_out) d0 = p.kv_out + t * row + at;
      if (p.cache) {
        const int64_t slot = p.slot_mapping[t];
        if (slot >= 0 && slot < p.num_slots) d1 = p.cache + slot * row + at;
      }
    }
#pragma unroll
    for (int k = 0; k < kCh; ++k) {
      const int c = (k * L + lane) * V;
      if (!on || c >= n) continue;
      if (!is_v && weight) {
        if constexpr (V == 8) {
          float w[8];
          Vec<T, 8>::load(weight + c, w);
#pragma unroll
          for (int e = 0; e < 8; ++e) x[k][e] *= rs * w[e];
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e)
            if (c + e < n) x[k][e] = x[k][e] * rs * Elem<T>::to_f(weight[c + e]);
        }
      }
      turn_pairs<V>(x[k], c, dims, co + pos * (dims / 2), si + pos * (dims / 2));
#pragma unroll
      for (int e = 0; e < V; ++e) x[k][e] *= f;
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        T* d = w == 0 ? d0 : d1;
        if (!d) continue;
        if constexpr (V == 8) {
          Vec<T, V>::store(d + c, x[k]);
        } else {
          d[c] = Elem<T>::from_f(x[k][0]);
          if (c + 1 < n) d[c + 1] = Elem<T>::from_f(x[k][1]);
        }
      }
    }
  }
}

template <typename T> struct WindowParams {
  T* out;                                    // (tokens, heads * vdim)
  const T* q; int64_t q_stride;              // (tokens, heads * dim)
  const T* cache;                            // (blocks, block_size, kv_heads * (dim + vdim))
  const int32_t* tables; int64_t bt_stride; int max_blocks, block_size; int64_t num_blocks;
  const int32_t* cu_q; int num_seqs;
  const int64_t* positions;
  const float* bias; int64_t bias_stride; int distances;       // bias[h * bias_stride + distance]
  const T* sink;
  int heads, kv_heads, dim, vdim;
  int64_t window;
  float scale;
  const float2* turn; int64_t table_rows;                      // (vdim / 2, table_rows) cos, sin: results are turned back; null: not
  // rows only
  float cap; const float *r1, *r2;           // cap > 0: score = cap tanh(score / cap) - r1[h] ln(1 + r2[h] distance)
  int cross;                                 // value heads of which every head's result is wanted: out (tokens, heads, cross, vdim); 0: its own
  int maps; int64_t chunk;                   // key heads per value head (query heads: [head][map]); chunk > 0: positions see their own chunk
  float* out_f;                              // fp32 results instead of out
  // decode
  const T* gate; int64_t gate_stride; float lambda, mult, eps;   // two maps: their difference, normed, times mult and sigmoid(gate)
  int splits;
  float *part_ml, *part_o;                   // (batch, splits, heads, 2) and (.., vdim)
};

constexpr int kWaThreads = 256, kWaHeads = 4, kWaKeys = 32, kWaPer = 4;    // vdim up to kWaThreads * kWaPer

template <typename T>
__global__ void __launch_bounds__(kWaThreads) window_attention_rows_kernel(const WindowParams<T> p) {
  extern __shared__ __align__(16) float sm[];
  const int group = p.heads / p.kv_heads, chunks = (group + kWaHeads - 1) / kWaHeads;
  const int kv = blockIdx.y / chunks, g0 = (blockIdx.y - kv * chunks) * kWaHeads;
  const int nh = min(kWaHeads, group - g0);
  const int D = p.dim, VD = p.vdim, v_heads = p.kv_heads / p.maps, row = p.kv_heads * D + v_heads * VD;
  const int vh = p.cross ? blockIdx.z : kv / p.maps;
  // query heads over key head kv: one per head of the group, `maps` apart
  auto head_at = [&](int i) { return (kv / p.maps * group + g0 + i) * p.maps + kv % p.maps; };
  float* sq = sm;                               // [kWaHeads][D]
  float* sk = sq + kWaHeads * D;                // [kWaKeys][D + 1]
  float* sv = sk + kWaKeys * (D + 1);           // [kWaKeys][VD]
  float* ss = sv + kWaKeys * VD;                // [kWaHeads][kWaKeys]
  __shared__ float s_m[kWaHeads], s_l[kWaHeads], s_c[kWaHeads];
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = seq_of_token(p.cu_q, p.num_seqs, t);
  const int32_t* table = p.tables + static_cast<int64_t>(seq) * p.bt_stride;
  const int64_t pos = p.positions[t];
  const int nk = static_cast<int>(min(pos + 1, static_cast<int64_t>(p.max_blocks) * p.block_size));
  const int first = static_cast<int>(max(p.chunk ? pos / p.chunk * p.chunk : pos - p.window + 1, static_cast<int64_t>(0)));
  for (int i = tid; i < kWaHeads * D; i += kWaThreads) {
    const int h = i / D, j = i - h * D;
    sq[i] = h < nh ? Elem<T>::to_f(p.q[t * p.q_stride + static_cast<int64_t>(head_at(h)) * D + j]) : 0.f;
  }
  // the sink is one more score without a value: it opens the running maximum and sum
  if (tid < kWaHeads) {
    s_m[tid] = tid < nh && p.sink ? Elem<T>::to_f(p.sink[head_at(tid)]) : -INFINITY;
    s_l[tid] = tid < nh && p.sink ? 1.f : 0.f;
  }
  float acc[kWaHeads][kWaPer];
#pragma unroll
  for (int h = 0; h < kWaHeads; ++h)
#pragma unroll
    for (int i = 0; i < kWaPer; ++i) acc[h][i] = 0.f;

  for (int k0 = first; k0 < nk; k0 += kWaKeys) {
    __syncthreads();
    for (int k = warp; k < kWaKeys; k += kWaThreads / 32) {
      const int at = k0 + k, blk = at / p.block_size;
      const int32_t phys = at < nk && blk < p.max_blocks ? table[blk] : -1;
      const bool ok = phys >= 0 && phys < p.num_blocks;
      const T* src = p.cache + (static_cast<int64_t>(ok ? phys : 0) * p.block_size + (at - blk * p.block_size)) * row;
      for (int i = lane; i < D; i += 32) sk[k * (D + 1) + i] = ok ? Elem<T>::to_f(src[kv * D + i]) : 0.f;
      for (int i = lane; i < VD; i += 32) sv[k * VD + i] = ok ? Elem<T>::to_f(src[p.kv_heads * D + vh * VD + i]) : 0.f;
      if (lane < kWaHeads) {
        float b = ok ? 0.f : -INFINITY;
        if (ok && p.bias && lane < nh)
          b = p.bias[head_at(lane) * p.bias_stride + min(static_cast<int>(pos) - at, p.distances - 1)];
        if (ok && p.r1 && lane < nh) b = -p.r1[head_at(lane)] * log1pf(p.r2[head_at(lane)] * static_cast<float>(static_cast<int>(pos) - at));
        ss[lane * kWaKeys + k] = b;
      }
    }
    __syncthreads();
    {  // two threads per (head, key)
      const int pair = tid >> 1, h = pair / kWaKeys, k = pair % kWaKeys, half = tid & 1;
      const float *a = sq + h * D, *b = sk + k * (D + 1);
      float s = 0.f;
      for (int i = half; i < D; i += 2) s = fmaf(a[i], b[i], s);
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s *= p.scale;
      if (p.cap > 0.f) s = p.cap * tanhf(s / p.cap);
      if (half == 0) ss[h * kWaKeys + k] += s;     // -inf stays -inf
    }
    __syncthreads();
    if (warp < kWaHeads) {
      const float s = ss[warp * kWaKeys + lane];
      float mx = s;
#pragma unroll
      for (int o = 16; o; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_old = s_m[warp], m_new = fmaxf(m_old, mx);
      const float pr = m_new == -INFINITY ? 0.f : expf(s - m_new);
      const float sum = warp_sum(pr);
      ss[warp * kWaKeys + lane] = pr;
      if (lane == 0) {
        const float corr = m_new == -INFINITY ? 1.f : expf(m_old - m_new);
        s_c[warp] = corr;
        s_l[warp] = s_l[warp] * corr + sum;
        s_m[warp] = m_new;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kWaPer; ++i) {
      const int d = tid + i * kWaThreads;
      if (d < VD) {
#pragma unroll
        for (int h = 0; h < kWaHeads; ++h) acc[h][i] *= s_c[h];
        for (int k = 0; k < kWaKeys; ++k) {
          const float v = sv[k * VD + d];
#pragma unroll
          for (int h = 0; h < kWaHeads; ++h) acc[h][i] = fmaf(ss[h * kWaKeys + k], v, acc[h][i]);
        }
      }
    }
  }
  __syncthreads();
  const int64_t angle = p.turn ? table_row(pos, p.table_rows) : 0;
#pragma unroll
  for (int h = 0; h < kWaHeads; ++h) {
    if (h >= nh) break;
    const float l = s_l[h], inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
    for (int i = 0; i < kWaPer; ++i) {
      const int d = tid + i * kWaThreads;
      if (p.turn && i * kWaThreads < VD) {      // the other column of the pair is the neighbouring thread's
        const float other = __shfl_xor_sync(0xffffffffu, acc[h][i], 1);
        if (d < VD) {
          const float2 cs = p.turn[d / 2 * p.table_rows + angle];
          acc[h][i] = fmaf(acc[h][i], cs.x, d & 1 ? -other * cs.y : other * cs.y);
        }
      }
      if (d < VD) {
        const int64_t at = (p.cross ? (static_cast<int64_t>(t) * p.heads + head_at(h)) * p.cross + vh : static_cast<int64_t>(t) * p.heads + head_at(h)) * VD + d;
        if (p.out_f) p.out_f[at] = acc[h][i] * inv;
        else p.out[at] = Elem<T>::from_f(acc[h][i] * inv);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ decode
// One CTA per (piece of the window, KV head and tile of 16 query heads, sequence): four warps stream 16-key tiles of
// their own through cp.async rings; the query heads are the rows of m16n8k16 products.  Attention weights enter their
// product as value and rounding residue.
//
// MAPS = 2: every head has two maps, with queries and keys of their own and the same values.  The upper eight rows are the
// heads' first maps, the lower eight the second ones; the rows of the other map are left out of each product with keys.
constexpr int kWdWarps = 4, kWdThreads = 32 * kWdWarps, kWdStages = 3, kWdTile = 16;
constexpr float kWdNeg = -1e30f;

template <int KD, int VD, int MAPS = 1> struct WdShape {
  static constexpr int kK = MAPS * kWdTile * KD * 2, kV = kWdTile * VD * 2, kStage = kK + kV, kWarp = kWdStages * kStage;
  static constexpr int kRing = kWdWarps * kWarp, kStride = VD + 8;
  static constexpr int kMerge = kWdWarps * 16 * (kStride + 2) * 4;
  static constexpr int kSmem = kRing > kMerge ? kRing : kMerge;
};

// What becomes of the two maps' results of a row: a1 - lambda a2, its RMS norm over the head, factor and gate.  One warp;
// get(d) gives the difference in columns d and d + 1.
template <typename T, typename F>
__device__ __forceinline__ void diff_finish(const WindowParams<T>& p, int64_t row, int h, int lane, F&& get) {
  constexpr int kHold = 4;               // vdim up to 256
  float2 o[kHold];
  float acc = 0.f;
#pragma unroll
  for (int i = 0; i < kHold; ++i) {
    const int d = (i * 32 + lane) * 2;
    o[i] = d < p.vdim ? get(d) : make_float2(0.f, 0.f);
    acc = fmaf(o[i].x, o[i].x, fmaf(o[i].y, o[i].y, acc));
  }
  const float f = p.mult / sqrtf(warp_sum(acc) / static_cast<float>(p.vdim) + p.eps);
#pragma unroll
  for (int i = 0; i < kHold; ++i) {
    const int d = (i * 32 + lane) * 2;
    if (d >= p.vdim) continue;
    const T *g = p.gate + row * p.gate_stride + static_cast<int64_t>(h) * p.vdim + d;
    T* out = p.out + (row * p.heads + h) * p.vdim + d;
    out[0] = Elem<T>::from_f(o[i].x * f * sigmoid_t<T>(Elem<T>::to_f(g[0])));
    out[1] = Elem<T>::from_f(o[i].y * f * sigmoid_t<T>(Elem<T>::to_f(g[1])));
  }
}

template <int KD, int VD, int MAPS>
__global__ void __launch_bounds__(kWdThreads, MAPS * KD + VD > 256 ? 1 : 2)
window_decode_kernel(const WindowParams<__nv_bfloat16> p) {
  using T = __nv_bfloat16;
  using S = WdShape<KD, VD, MAPS>;
  constexpr int R = 16 / MAPS;           // heads per tile of rows
  using Mma = Mma16816<T>;
  constexpr int KSTEPS = KD / 16, NT = VD / 8, KC = KD / 8, VC = VD / 8;
  extern __shared__ __align__(128) unsigned char smem[];
  __shared__ uint32_t s_mask[kWdWarps][kWdStages];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int group = p.heads / p.kv_heads, mtiles = (group + R - 1) / R;
  const int kv = blockIdx.y / mtiles, mt = blockIdx.y - kv * mtiles, b = blockIdx.z, split = blockIdx.x;
  const int rows = min(R, group - mt * R), h0 = kv * group + mt * R;
  const int64_t pos64 = p.positions[b];
  const int pos = static_cast<int>(pos64);
  const int nk = static_cast<int>(min(pos64 + 1, static_cast<int64_t>(p.max_blocks) * p.block_size));
  const int lo = static_cast<int>(max(MAPS > 1 ? pos64 / p.chunk * p.chunk : pos64 - p.window + 1, static_cast<int64_t>(0)));
  const int span = max(nk - lo, 0);
  const int len = ((span + p.splits - 1) / p.splits + kWdTile - 1) / kWdTile * kWdTile;
  const int k_begin = lo + split * len, k_end = min(k_begin + len, nk);
  const int tiles = k_end > k_begin ? (k_end - k_begin + kWdTile - 1) / kWdTile : 0;
  const int my_tiles = tiles > warp ? (tiles - warp + kWdWarps - 1) / kWdWarps : 0;
  const int32_t* table = p.tables + static_cast<int64_t>(b) * p.bt_stride;
  const int64_t row_elems = static_cast<int64_t>(p.kv_heads) * (MAPS * p.dim + p.vdim);
  const T *k_base = p.cache + kv * MAPS * p.dim, *v_base = p.cache + p.kv_heads * MAPS * p.dim + kv * p.vdim;
  const uint32_t ring = smem_u32(smem) + warp * S::kWarp;
  const int kc_real = p.dim / 8, vc_real = p.vdim / 8;

  auto issue = [&](int i) {
    if (i < my_tiles) {
      const int stage = i % kWdStages, tok0 = k_begin + (i * kWdWarps + warp) * kWdTile;
      const int me = tok0 + (lane & 15), blk = me / p.block_size;
      int64_t at = -1;
      if (me < k_end && blk < p.max_blocks) {
        const int32_t phys = __ldg(table + blk);
        if (phys >= 0 && phys < p.num_blocks) at = (static_cast<int64_t>(phys) * p.block_size + (me - blk * p.block_size)) * row_elems;
      }
      const uint32_t live = __ballot_sync(0xffffffffu, at >= 0) & 0xffffu;
      if (lane == 0) s_mask[warp][stage] = live;
      const uint32_t kd = ring + stage * S::kStage, vd = kd + S::kK;
#pragma unroll
      for (int c0 = 0; c0 < MAPS * kWdTile * KC; c0 += 32) {
        const int m = c0 / (kWdTile * KC), r = (c0 + lane) / KC % kWdTile, c = (c0 + lane) % KC;
        const int64_t src = __shfl_sync(0xffffffffu, at, r);
        const bool ok = src >= 0 && c < kc_real;
        cp_async16(kd + (m * kWdTile + r) * (KD * 2) + ((c ^ (r & 7)) << 4), ok ? k_base + src + m * p.dim + c * 8 : p.cache, ok ? 16 : 0);
      }
#pragma unroll
      for (int c0 = 0; c0 < kWdTile * VC; c0 += 32) {
        const int r = (c0 + lane) / VC, c = (c0 + lane) % VC;
        const int64_t src = __shfl_sync(0xffffffffu, at, r);
        const bool ok = src >= 0 && c < vc_real;
        cp_async16(vd + r * (VD * 2) + ((c ^ (r & 7)) << 4), ok ? v_base + src + c * 8 : p.cache, ok ? 16 : 0);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int i = 0; i < kWdStages - 1; ++i) issue(i);

  uint32_t qa[KSTEPS][4];
  {
    const T* qb = p.q + b * p.q_stride + static_cast<int64_t>(h0) * MAPS * p.dim;
    const bool v0 = g < rows, v1 = MAPS > 1 ? v0 : g + 8 < rows;
    const uint32_t* q0 = reinterpret_cast<const uint32_t*>(qb + static_cast<int64_t>(MAPS * g) * p.dim);
    const uint32_t* q1 = reinterpret_cast<const uint32_t*>(qb + static_cast<int64_t>(MAPS > 1 ? 2 * g + 1 : g + 8) * p.dim);
    const int half = p.dim / 2;
#pragma unroll
    for (int ks = 0; ks < KSTEPS; ++ks) {
      const int c = ks * 8 + t;
      qa[ks][0] = v0 && c < half ? __ldg(q0 + c) : 0u;
      qa[ks][1] = v1 && c < half ? __ldg(q1 + c) : 0u;
      qa[ks][2] = v0 && c + 4 < half ? __ldg(q0 + c + 4) : 0u;
      qa[ks][3] = v1 && c + 4 < half ? __ldg(q1 + c + 4) : 0u;
    }
  }
  const float scale2 = p.scale * 1.4426950408889634f;
  const float* bias0 = p.bias ? p.bias + (h0 + min(g, rows - 1)) * p.bias_stride : nullptr;
  const float* bias1 = p.bias ? p.bias + (h0 + min(g + 8, rows - 1)) * p.bias_stride : nullptr;
  const float far0 = bias0 ? bias0[p.distances - 1] * 1.4426950408889634f : 0.f;
  const float far1 = bias1 ? bias1[p.distances - 1] * 1.4426950408889634f : 0.f;

  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m0 = kWdNeg, m1 = kWdNeg, l0 = 0.f, l1 = 0.f;
  for (int i = 0; i < my_tiles; ++i) {
    cp_async_wait<kWdStages - 2>();
    __syncwarp();
    const int stage = i % kWdStages, tok0 = k_begin + (i * kWdWarps + warp) * kWdTile;
    const uint32_t kd = ring + stage * S::kStage, vd = kd + S::kK;
    const uint32_t live = s_mask[warp][stage];
    float s[2][4] = {};
    {
      const int row = (lane & 7) + ((lane >> 4) << 3), csel = (lane >> 3) & 1;
#pragma unroll
      for (int ks = 0; ks < KSTEPS; ++ks) {
        uint32_t kb[4];
        ldmatrix_x4(kb, kd + row * (KD * 2) + (((2 * ks + csel) ^ (row & 7)) << 4));
        Mma::run(s[0], qa[ks], kb[0], kb[1]);
        Mma::run(s[1], qa[ks], kb[2], kb[3]);
      }
      if constexpr (MAPS > 1) {
        float s2[2][4] = {};
#pragma unroll
        for (int ks = 0; ks < KSTEPS; ++ks) {
          uint32_t kb[4];
          ldmatrix_x4(kb, kd + (kWdTile + row) * (KD * 2) + (((2 * ks + csel) ^ (row & 7)) << 4));
          Mma::run(s2[0], qa[ks], kb[0], kb[1]);
          Mma::run(s2[1], qa[ks], kb[2], kb[3]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) { s[n][2] = s2[n][2]; s[n][3] = s2[n][3]; }
      }
    }
    issue(i + kWdStages - 1);
    const bool far = pos - tok0 - (kWdTile - 1) >= p.distances - 1;      // every key of the tile has the last bias
    float mx0 = kWdNeg, mx1 = kWdNeg;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int col = n * 8 + 2 * t + e;
        float b0 = far0, b1 = far1;
        if (p.bias && !far) {
          const int d = min(max(pos - tok0 - col, 0), p.distances - 1);
          b0 = __ldg(bias0 + d) * 1.4426950408889634f;
          b1 = __ldg(bias1 + d) * 1.4426950408889634f;
        }
        const bool ok = (live >> col) & 1u;
        s[n][e] = ok ? fmaf(s[n][e], scale2, b0) : -INFINITY;
        s[n][2 + e] = ok ? fmaf(s[n][2 + e], scale2, b1) : -INFINITY;
      }
      mx0 = fmaxf(mx0, fmaxf(s[n][0], s[n][1]));
      mx1 = fmaxf(mx1, fmaxf(s[n][2], s[n][3]));
    }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1), a0 = fast_exp2(m0 - mn0), a1 = fast_exp2(m1 - mn1);
    m0 = mn0;
    m1 = mn1;
    float ps0 = 0.f, ps1 = 0.f;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      s[n][0] = fast_exp2(s[n][0] - mn0); s[n][1] = fast_exp2(s[n][1] - mn0);
      s[n][2] = fast_exp2(s[n][2] - mn1); s[n][3] = fast_exp2(s[n][3] - mn1);
      ps0 += s[n][0] + s[n][1];
      ps1 += s[n][2] + s[n][3];
    }
    l0 = l0 * a0 + ps0;
    l1 = l1 * a1 + ps1;
    uint32_t pa[4], pl[4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        pa[2 * n + hh] = pack2<T>(s[n][2 * hh], s[n][2 * hh + 1]);
        const float2 hi = Elem<T>::to_f2(*reinterpret_cast<const __nv_bfloat162*>(&pa[2 * n + hh]));
        pl[2 * n + hh] = pack2<T>(s[n][2 * hh] - hi.x, s[n][2 * hh + 1] - hi.y);
      }
    if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
      for (int j = 0; j < NT; ++j) { o[j][0] *= a0; o[j][1] *= a0; o[j][2] *= a1; o[j][3] *= a1; }
    }
    {
      const int row = (lane & 7) + (((lane >> 3) & 1) << 3), csel = lane >> 4;
#pragma unroll
      for (int jp = 0; jp < NT / 2; ++jp) {
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, vd + row * (VD * 2) + (((2 * jp + csel) ^ (row & 7)) << 4));
        Mma::run(o[2 * jp], pa, vb[0], vb[1]);
        Mma::run(o[2 * jp + 1], pa, vb[2], vb[3]);
        Mma::run(o[2 * jp], pl, vb[0], vb[1]);
        Mma::run(o[2 * jp + 1], pl, vb[2], vb[3]);
      }
    }
    __syncwarp();
  }
  cp_async_wait<0>();
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  __syncthreads();                       // the rings are idle
  float* sO = reinterpret_cast<float*>(smem);
  float* sML = sO + kWdWarps * 16 * S::kStride;
  {
    float* mine = sO + warp * 16 * S::kStride;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      *reinterpret_cast<float2*>(mine + g * S::kStride + j * 8 + 2 * t) = make_float2(o[j][0], o[j][1]);
      *reinterpret_cast<float2*>(mine + (g + 8) * S::kStride + j * 8 + 2 * t) = make_float2(o[j][2], o[j][3]);
    }
    if (t == 0) {
      sML[(warp * 16 + g) * 2] = m0;
      sML[(warp * 16 + g) * 2 + 1] = l0;
      sML[(warp * 16 + g + 8) * 2] = m1;
      sML[(warp * 16 + g + 8) * 2 + 1] = l1;
    }
  }
  __syncthreads();
  if constexpr (MAPS > 1) {
    auto scales = [&](int r, float (&f)[kWdWarps], float& M) {     // factors of the warps' parts of a row; returns its sum
      M = kWdNeg;
#pragma unroll
      for (int w = 0; w < kWdWarps; ++w) M = fmaxf(M, sML[(w * 16 + r) * 2]);
      float L = 0.f;
#pragma unroll
      for (int w = 0; w < kWdWarps; ++w) {
        f[w] = fast_exp2(sML[(w * 16 + r) * 2] - M);
        L = fmaf(f[w], sML[(w * 16 + r) * 2 + 1], L);
      }
      return L;
    };
    auto joined = [&](int r, const float (&f)[kWdWarps], int d) {
      float2 acc = make_float2(0.f, 0.f);
#pragma unroll
      for (int w = 0; w < kWdWarps; ++w) {
        const float2 o2 = *reinterpret_cast<const float2*>(sO + (w * 16 + r) * S::kStride + d);
        acc.x = fmaf(f[w], o2.x, acc.x);
        acc.y = fmaf(f[w], o2.y, acc.y);
      }
      return acc;
    };
    for (int r = warp; r < rows; r += kWdWarps) {
      float f1[kWdWarps], f2[kWdWarps], M1, M2;
      const float L1 = scales(r, f1, M1), L2 = scales(r + 8, f2, M2);
      if (p.splits == 1) {
        const float i1 = L1 > 0.f ? 1.f / L1 : 0.f, i2 = L2 > 0.f ? p.lambda / L2 : 0.f;
        diff_finish(p, b, h0 + r, lane, [&](int d) {
          const float2 a1 = joined(r, f1, d), a2 = joined(r + 8, f2, d);
          return make_float2(a1.x * i1 - a2.x * i2, a1.y * i1 - a2.y * i2);
        });
      } else {
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          const int64_t pi = ((static_cast<int64_t>(b) * p.splits + split) * p.heads + h0 + r) * 2 + m;
          for (int d = lane * 2; d < p.vdim; d += 64)
            *reinterpret_cast<float2*>(p.part_o + pi * p.vdim + d) = m ? joined(r + 8, f2, d) : joined(r, f1, d);
          if (lane == 0) {
            p.part_ml[pi * 2] = m ? M2 : M1;
            p.part_ml[pi * 2 + 1] = m ? L2 : L1;
          }
        }
      }
    }
    return;
  }
  const int half = p.vdim / 2;           // a thread has pairs of neighbouring columns
  const int64_t angle = p.turn ? table_row(pos64, p.table_rows) : 0;
  for (int i = tid; i < rows * half; i += kWdThreads) {
    const int r = i / half, d = (i - r * half) * 2, h = h0 + r;
    float M = kWdNeg;
#pragma unroll
    for (int w = 0; w < kWdWarps; ++w) M = fmaxf(M, sML[(w * 16 + r) * 2]);
    const float sk = p.sink ? __bfloat162float(p.sink[h]) * 1.4426950408889634f : kWdNeg;
    if (p.splits == 1 && p.sink) M = fmaxf(M, sk);
    float2 acc = make_float2(0.f, 0.f);
    float L = p.splits == 1 && p.sink ? fast_exp2(sk - M) : 0.f;
#pragma unroll
    for (int w = 0; w < kWdWarps; ++w) {
      const float f = fast_exp2(sML[(w * 16 + r) * 2] - M);
      const float2 o2 = *reinterpret_cast<const float2*>(sO + (w * 16 + r) * S::kStride + d);
      acc.x = fmaf(f, o2.x, acc.x);
      acc.y = fmaf(f, o2.y, acc.y);
      L = fmaf(f, sML[(w * 16 + r) * 2 + 1], L);
    }
    if (p.splits == 1) {
      const float inv = L > 0.f ? 1.f / L : 0.f;
      acc.x *= inv;
      acc.y *= inv;
      if (p.turn) turn_back(acc.x, acc.y, p.turn[d / 2 * p.table_rows + angle]);
      *reinterpret_cast<__nv_bfloat162*>(p.out + (static_cast<int64_t>(b) * p.heads + h) * p.vdim + d) = __floats2bfloat162_rn(acc.x, acc.y);
    } else {
      const int64_t pi = (static_cast<int64_t>(b) * p.splits + split) * p.heads + h;
      *reinterpret_cast<float2*>(p.part_o + pi * p.vdim + d) = acc;
      if (d == 0) {
        p.part_ml[pi * 2] = M;
        p.part_ml[pi * 2 + 1] = L;
      }
    }
  }
}

// Joins the pieces of a sequence and head, and adds the sink.
__global__ void __launch_bounds__(128) window_join_kernel(const WindowParams<__nv_bfloat16> p) {
  const int h = blockIdx.x, b = blockIdx.y;
  const int64_t first = static_cast<int64_t>(b) * p.splits * p.heads + h;
  float M = p.sink ? __bfloat162float(p.sink[h]) * 1.4426950408889634f : kWdNeg;
  float L = p.sink ? 1.f : 0.f;
  const float opened = M;
  for (int s = 0; s < p.splits; ++s) M = fmaxf(M, p.part_ml[(first + static_cast<int64_t>(s) * p.heads) * 2]);
  L *= fast_exp2(opened - M);
  for (int s = 0; s < p.splits; ++s) {
    const float* ml = p.part_ml + (first + static_cast<int64_t>(s) * p.heads) * 2;
    L = fmaf(fast_exp2(ml[0] - M), ml[1], L);
  }
  const float inv = L > 0.f ? 1.f / L : 0.f;
  const int64_t angle = p.turn ? table_row(p.positions[b], p.table_rows) : 0;
  for (int d = threadIdx.x * 2; d < p.vdim; d += 256) {
    float2 acc = make_float2(0.f, 0.f);
    for (int s = 0; s < p.splits; ++s) {
      const int64_t pi = first + static_cast<int64_t>(s) * p.heads;
      const float f = fast_exp2(p.part_ml[pi * 2] - M);
      const float2 o2 = *reinterpret_cast<const float2*>(p.part_o + pi * p.vdim + d);
      acc.x = fmaf(f, o2.x, acc.x);
      acc.y = fmaf(f, o2.y, acc.y);
    }
    acc.x *= inv;
    acc.y *= inv;
    if (p.turn) turn_back(acc.x, acc.y, p.turn[d / 2 * p.table_rows + angle]);
    *reinterpret_cast<__nv_bfloat162*>(p.out + (static_cast<int64_t>(b) * p.heads + h) * p.vdim + d) = __floats2bfloat162_rn(acc.x, acc.y);
  }
}

// The same for two maps: a warp per sequence and head.
__global__ void __launch_bounds__(128) diff_join_kernel(const WindowParams<__nv_bfloat16> p, int batch) {
  const int i = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31, b = i / p.heads, h = i - b * p.heads;
  if (b >= batch) return;
  const int64_t first = (static_cast<int64_t>(b) * p.splits * p.heads + h) * 2, step = static_cast<int64_t>(p.heads) * 2;
  float M[2] = {kWdNeg, kWdNeg}, L[2] = {0.f, 0.f};
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    for (int s = 0; s < p.splits; ++s) M[m] = fmaxf(M[m], p.part_ml[(first + s * step + m) * 2]);
    for (int s = 0; s < p.splits; ++s) {
      const float* ml = p.part_ml + (first + s * step + m) * 2;
      L[m] = fmaf(fast_exp2(ml[0] - M[m]), ml[1], L[m]);
    }
  }
  const float i1 = L[0] > 0.f ? 1.f / L[0] : 0.f, i2 = L[1] > 0.f ? p.lambda / L[1] : 0.f;
  diff_finish(p, b, h, lane, [&](int d) {
    float2 acc = make_float2(0.f, 0.f);
    for (int s = 0; s < p.splits; ++s) {
      const int64_t pi = first + s * step;
      const float f1 = fast_exp2(p.part_ml[pi * 2] - M[0]) * i1, f2 = fast_exp2(p.part_ml[pi * 2 + 2] - M[1]) * i2;
      const float2 a1 = *reinterpret_cast<const float2*>(p.part_o + pi * p.vdim + d), a2 = *reinterpret_cast<const float2*>(p.part_o + (pi + 1) * p.vdim + d);
      acc.x += f1 * a1.x - f2 * a2.x;
      acc.y += f1 * a1.y - f2 * a2.y;
    }
    return acc;
  });
}

// Difference, norm and gate for results in fp32, (tokens, heads, 2, vdim): a warp per token and head.
template <typename T> struct DiffParams {
  T* out; const float* a; const T* gate; int64_t gate_stride; int64_t tokens; int heads, vdim; float lambda, mult, eps;
};
template <typename T> __global__ void __launch_bounds__(256) diff_norm_gate_kernel(const DiffParams<T> p) {
  const int lane = threadIdx.x & 31;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5); i < p.tokens * p.heads; i += static_cast<int64_t>(gridDim.x) * 8) {
    const int64_t t = i / p.heads, h = i - t * p.heads;
    const float *a1 = p.a + i * 2 * p.vdim, *a2 = a1 + p.vdim;
    float acc = 0.f;
    for (int d = lane; d < p.vdim; d += 32) {
      const float o = a1[d] - p.lambda * a2[d];
      acc = fmaf(o, o, acc);
    }
    const float f = p.mult / sqrtf(warp_sum(acc) / static_cast<float>(p.vdim) + p.eps);
    const T* g = p.gate + t * p.gate_stride + h * p.vdim;
    for (int d = lane; d < p.vdim; d += 32)
      p.out[i * p.vdim + d] = Elem<T>::from_f((a1[d] - p.lambda * a2[d]) * f * sigmoid_t<T>(Elem<T>::to_f(g[d])));
  }
}

template <int KD, int VD, int MAPS = 1> static int launch_window_decode(const WindowParams<__nv_bfloat16>& p, int batch, cudaStream_t st) {
  const int smem = WdShape<KD, VD, MAPS>::kSmem;
  const cudaError_t e = cudaFuncSetAttribute(window_decode_kernel<KD, VD, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return fail(MV_ERR_CUDA, "window_decode: %s", cudaGetErrorString(e));
  const int mtiles = (p.heads / p.kv_heads + 16 / MAPS - 1) / (16 / MAPS);
  window_decode_kernel<KD, VD, MAPS><<<dim3(p.splits, p.kv_heads * mtiles, batch), kWdThreads, smem, st>>>(p);
  int rc = check_launch("window_decode");
  if (rc || p.splits == 1) return rc;
  if (MAPS > 1) diff_join_kernel<<<static_cast<unsigned>((static_cast<int64_t>(batch) * p.heads + 3) / 4), 128, 0, st>>>(p, batch);
  else window_join_kernel<<<dim3(p.heads, batch), 128, 0, st>>>(p);
  return check_launch("window_join");
}

// Pieces per sequence: enough CTAs to fill the GPU twice, none of less than 64 keys.  Depends on shapes only.
static int window_splits(int batch, int heads, int kv_heads, int64_t most_keys, int rows = 16) {
  const int64_t units = static_cast<int64_t>(batch) * kv_heads * ((heads / kv_heads + rows - 1) / rows);
  const int64_t want = (2 * kNumSMs + units - 1) / std::max<int64_t>(units, 1);
  return static_cast<int>(std::max<int64_t>(1, std::min<int64_t>({want, most_keys / 64, 64})));
}

static bool check_turn(const float* turn, int64_t table_rows, int vdim) {
  return !turn || (table_rows > 0 && vdim % 2 == 0 && (reinterpret_cast<uintptr_t>(turn) & 7u) == 0);
}
static int check_window(const char* what, int heads, int kv_heads, int dim, int vdim, int64_t window, int block_size) {
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || window <= 0 || block_size <= 0)
    return fail(MV_ERR_SHAPE, "%s: heads %d over %d, dim %d, vdim %d, window %lld", what, heads, kv_heads, dim, vdim, static_cast<long long>(window));
  return MV_OK;
}

}  // namespace mv

extern "C" int mv_kv_norm_store(void* q, const void* k, const void* v, int64_t stride, const void* q_weight,
                                const void* k_weight, void* kv_out, void* cache, const int64_t* slot_mapping,
                                int64_t num_slots, int64_t tokens, int q_rows, int k_rows, int v_rows, float eps, int dtype,
                                void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "kv_norm_store: dtype %d", dtype);
  if (tokens < 0 || q_rows <= 0 || k_rows <= 0 || v_rows <= 0) return fail(MV_ERR_SHAPE, "kv_norm_store: %d, %d, %d rows", q_rows, k_rows, v_rows);
  if (tokens == 0) return MV_OK;
  if (!q || !k || !v || !q_weight || !k_weight || (cache && !slot_mapping)) return fail(MV_ERR_NULL, "kv_norm_store: null pointer");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int eb = sizeof(T);
    auto go = [&](auto kernel) {
      kernel<<<static_cast<unsigned>(tokens), kKnThreads, 0, static_cast<cudaStream_t>(stream)>>>(
          static_cast<T*>(q), static_cast<const T*>(k), static_cast<const T*>(v), stride, static_cast<const T*>(q_weight),
          static_cast<const T*>(k_weight), static_cast<T*>(kv_out), static_cast<T*>(cache), slot_mapping, num_slots, q_rows,
          k_rows, v_rows, eps);
      return check_launch("kv_norm_store");
    };
    if (q_rows % 8 == 0 && k_rows % 8 == 0 && v_rows % 8 == 0 && vec8_ok(q, stride, eb) && vec8_ok(k, stride, eb) &&
        vec8_ok(v, stride, eb) && aligned16(q_weight) && aligned16(k_weight) && aligned16(kv_out) && aligned16(cache))
      return go(kv_norm_store_kernel<T, 8>);
    return go(kv_norm_store_kernel<T, 1>);
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_qkv_rope_store(void* q, const void* k, const void* v, int64_t stride, const void* q_weight,
                                 const void* k_weight, const void* temp, const float* cos_t, const float* sin_t, int dims,
                                 const float* vcos_t, const float* vsin_t, int64_t table_rows, const int64_t* positions,
                                 void* kv_out, void* cache, const int64_t* slot_mapping, int64_t num_slots, int64_t tokens,
                                 int heads, int kv_heads, int v_heads, int dim, int vdim, float eps, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "qkv_rope_store: dtype %d", dtype);
  if (tokens < 0 || heads < 0 || kv_heads < 0 || !kv_heads != !v_heads || v_heads < 0 || heads + kv_heads == 0 || dim <= 0 || vdim < 0 ||
      (kv_heads && vdim <= 0) || dims < 0 || dims > dim || dims % 2 || (vcos_t && vdim % 2) || table_rows <= 0)
    return fail(MV_ERR_SHAPE, "qkv_rope_store: heads %d over %d and %d, dim %d (%d rotated), vdim %d", heads, kv_heads, v_heads, dim, dims, vdim);
  const int widest = kv_heads ? std::max(dim, vdim) : dim;
  if (widest > 1024) return fail(MV_ERR_LIMIT, "qkv_rope_store: dim %d, vdim %d (at most 1024)", dim, vdim);
  const int64_t items = tokens * (heads + static_cast<int64_t>(kv_heads) + v_heads);
  if (items >= 1LL << 31) return fail(MV_ERR_LIMIT, "qkv_rope_store: %lld tokens", static_cast<long long>(tokens));
  if (tokens == 0) return MV_OK;
  if ((heads && (!q || !q_weight)) || !positions || (dims && (!cos_t || !sin_t)) || !vcos_t != !vsin_t ||
      (kv_heads && (!k || !v)) || (cache && !slot_mapping))
    return fail(MV_ERR_NULL, "qkv_rope_store: null pointer");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int eb = sizeof(T);
    auto c = [](const void* x) { return static_cast<const T*>(x); };
    RopeStoreParams<T> p{static_cast<T*>(q), c(k), c(v), stride, c(q_weight), c(k_weight), c(temp), cos_t, sin_t, dims, vcos_t, vsin_t,
                         table_rows, positions, static_cast<T*>(kv_out), static_cast<T*>(cache), slot_mapping, num_slots, tokens,
                         heads, kv_heads, v_heads, dim, vdim, eps};
    auto go = [&](auto kernel, int lanes) {
      const int64_t blocks = (items + kKnThreads / lanes - 1) / (kKnThreads / lanes);
      kernel<<<static_cast<unsigned>(std::min<int64_t>(blocks, kNumSMs * 64)), kKnThreads, 0, static_cast<cudaStream_t>(stream)>>>(p);
      return check_launch("qkv_rope_store");
    };
    const bool v8 = dim % 8 == 0 && vdim % 8 == 0 && vec8_ok(q, stride, eb) && vec8_ok(k, stride, eb) && vec8_ok(v, stride, eb) &&
                    aligned16(kv_out) && aligned16(cache) && aligned16(q_weight) && aligned16(k_weight) && aligned16(cos_t) &&
                    aligned16(sin_t) && aligned16(vcos_t) && aligned16(vsin_t);
    if (v8 && widest <= 64) return go(qkv_rope_store_kernel<T, 8, 8, 1>, 8);
    if (v8 && widest <= 128) return go(qkv_rope_store_kernel<T, 8, 16, 1>, 16);
    if (v8 && widest <= 256) return go(qkv_rope_store_kernel<T, 8, 32, 1>, 32);
    if (v8) return go(qkv_rope_store_kernel<T, 8, 32, 4>, 32);
    return go(qkv_rope_store_kernel<T, 2, 32, 16>, 32);
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

// What the forms of attention on the kernel for any sizes differ in.
struct RowsForm {
  const float* bias = nullptr; int64_t bias_stride = 0; int distances = 1; const void* sink = nullptr;
  const float* turn = nullptr; int64_t table_rows = 0;
  float cap = 0.f; const float *r1 = nullptr, *r2 = nullptr; int cross = 0, maps = 1; int64_t chunk = 0; float* out_f = nullptr;
};
static int attention_rows(const char* what, void* out, const void* q, int64_t q_stride, const void* cache,
                          const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size, int64_t num_blocks,
                          const int32_t* cu_q, int num_seqs, const int64_t* positions, int64_t tokens, int heads, int kv_heads,
                          int dim, int vdim, int64_t window, float scale, const RowsForm& f, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "%s: dtype %d", what, dtype);
  const int rc = check_window(what, heads, kv_heads, dim, vdim, window, block_size);
  if (rc) return rc;
  if (!check_turn(f.turn, f.table_rows, vdim)) return fail(MV_ERR_SHAPE, "%s: rotation of %d columns", what, vdim);
  if (vdim > kWaThreads * kWaPer) return fail(MV_ERR_LIMIT, "%s: vdim %d (at most %d)", what, vdim, kWaThreads * kWaPer);
  if (f.bias && f.distances <= 0) return fail(MV_ERR_SHAPE, "%s: %d distances", what, f.distances);
  if (tokens <= 0) return tokens < 0 ? fail(MV_ERR_SHAPE, "%s: tokens", what) : static_cast<int>(MV_OK);
  if (!(out || f.out_f) || !q || !cache || !block_tables || !positions) return fail(MV_ERR_NULL, "%s: null pointer", what);
  const size_t smem = sizeof(float) * (static_cast<size_t>(kWaHeads) * dim + static_cast<size_t>(kWaKeys) * (dim + 1 + vdim) + kWaHeads * kWaKeys);
  if (smem > 227 * 1024) return fail(MV_ERR_LIMIT, "%s: dim %d, vdim %d", what, dim, vdim);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const cudaError_t e = cudaFuncSetAttribute(window_attention_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
    WindowParams<T> p{};
    p.out = static_cast<T*>(out); p.q = static_cast<const T*>(q); p.q_stride = q_stride; p.cache = static_cast<const T*>(cache);
    p.tables = block_tables; p.bt_stride = bt_stride; p.max_blocks = max_blocks; p.block_size = block_size; p.num_blocks = num_blocks;
    p.cu_q = cu_q; p.num_seqs = num_seqs; p.positions = positions; p.bias = f.bias; p.bias_stride = f.bias_stride; p.distances = f.distances;
    p.sink = static_cast<const T*>(f.sink); p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.window = window; p.scale = scale;
    p.turn = reinterpret_cast<const float2*>(f.turn); p.table_rows = f.table_rows;
    p.cap = f.cap; p.r1 = f.r1; p.r2 = f.r2; p.cross = f.cross; p.maps = f.maps; p.chunk = f.chunk; p.out_f = f.out_f;
    const int chunks = (heads / kv_heads + kWaHeads - 1) / kWaHeads;
    window_attention_rows_kernel<T><<<dim3(static_cast<unsigned>(tokens), kv_heads * chunks, f.cross ? f.cross : 1), kWaThreads, smem, static_cast<cudaStream_t>(stream)>>>(p);
    return check_launch(what);
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_window_attention_rows(void* out, const void* q, int64_t q_stride, const void* cache,
                                        const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size,
                                        int64_t num_blocks, const int32_t* cu_q, int num_seqs, const int64_t* positions,
                                        const float* bias, int64_t bias_stride, int distances, const void* sink,
                                        const float* turn, int64_t table_rows, int64_t tokens, int heads, int kv_heads,
                                        int dim, int vdim, int64_t window, float scale, int dtype, void* stream) {
  RowsForm f;
  f.bias = bias; f.bias_stride = bias_stride; f.distances = distances; f.sink = sink; f.turn = turn; f.table_rows = table_rows;
  return attention_rows("window_attention_rows", out, q, q_stride, cache, block_tables, bt_stride, max_blocks, block_size, num_blocks, cu_q,
                        num_seqs, positions, tokens, heads, kv_heads, dim, vdim, window, scale, f, dtype, stream);
}

extern "C" int mv_talk_attention_rows(float* out, const void* q, int64_t q_stride, const void* cache,
                                      const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size,
                                      int64_t num_blocks, const int32_t* cu_q, int num_seqs, const int64_t* positions,
                                      const float* r1, const float* r2, float cap, int64_t tokens, int heads, int kv_heads,
                                      int dim, int vdim, float scale, int dtype, void* stream) {
  RowsForm f;
  if (!(cap > 0.f)) return mv::fail(MV_ERR_SHAPE, "talk_attention_rows: cap %f", cap);
  if (!r1 || !r2) return mv::fail(MV_ERR_NULL, "talk_attention_rows: null pointer");
  f.r1 = r1; f.r2 = r2; f.cap = cap; f.cross = kv_heads; f.out_f = out;
  return attention_rows("talk_attention_rows", nullptr, q, q_stride, cache, block_tables, bt_stride, max_blocks, block_size, num_blocks, cu_q,
                        num_seqs, positions, tokens, heads, kv_heads, dim, vdim, 1LL << 40, scale, f, dtype, stream);
}

extern "C" int mv_diff_attention_rows(float* out, const void* q, int64_t q_stride, const void* cache,
                                      const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size,
                                      int64_t num_blocks, const int32_t* cu_q, int num_seqs, const int64_t* positions,
                                      int64_t chunk, int64_t tokens, int heads, int kv_heads, int dim, int vdim, float scale,
                                      int dtype, void* stream) {
  RowsForm f;
  if (chunk <= 0) return mv::fail(MV_ERR_SHAPE, "diff_attention_rows: chunk %lld", static_cast<long long>(chunk));
  f.maps = 2; f.chunk = chunk; f.out_f = out;
  return attention_rows("diff_attention_rows", nullptr, q, q_stride, cache, block_tables, bt_stride, max_blocks, block_size, num_blocks, cu_q,
                        num_seqs, positions, tokens, 2 * heads, 2 * kv_heads, dim, vdim, 1LL << 40, scale, f, dtype, stream);
}

// Bytes of scratch, or -1 when the kernel does not take the sizes.
extern "C" int64_t mv_window_decode_workspace_bytes(int batch, int heads, int kv_heads, int dim, int vdim, int64_t most_keys) {
  using namespace mv;
  if (batch < 0 || batch > 65535 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || dim % 8 || vdim % 8 ||
      dim > 256 || vdim > 256 || most_keys <= 0)
    return -1;
  const int splits = window_splits(batch, heads, kv_heads, most_keys);
  return splits == 1 ? 0 : static_cast<int64_t>(batch) * splits * heads * (vdim + 2) * 4;
}

extern "C" int mv_window_decode(void* out, const void* q, int64_t q_stride, const void* cache, const int32_t* block_tables,
                                int64_t bt_stride, int max_blocks, int block_size, int64_t num_blocks,
                                const int64_t* positions, const float* bias, int64_t bias_stride, int distances,
                                const void* sink, const float* turn, int64_t table_rows, int batch, int heads,
                                int kv_heads, int dim, int vdim, int64_t window, float scale, void* workspace, int64_t workspace_bytes, void* stream) {
  using namespace mv;
  const int rc = check_window("window_decode", heads, kv_heads, dim, vdim, window, block_size);
  if (rc) return rc;
  const int64_t most = std::min<int64_t>(window, static_cast<int64_t>(max_blocks) * block_size);
  const int64_t need = mv_window_decode_workspace_bytes(batch, heads, kv_heads, dim, vdim, std::max<int64_t>(most, 1));
  if (!check_turn(turn, table_rows, vdim)) return fail(MV_ERR_SHAPE, "window_decode: rotation of %d columns", vdim);
  if (need < 0) return fail(MV_ERR_LIMIT, "window_decode: dim %d, vdim %d, batch %d", dim, vdim, batch);
  if (bias && distances <= 0) return fail(MV_ERR_SHAPE, "window_decode: %d distances", distances);
  if (batch == 0) return MV_OK;
  if (!out || !q || !cache || !block_tables || !positions) return fail(MV_ERR_NULL, "window_decode: null pointer");
  if (!aligned16(cache) || (reinterpret_cast<uintptr_t>(q) & 3u) || (reinterpret_cast<uintptr_t>(out) & 3u) || q_stride % 2)
    return fail(MV_ERR_ALIGN, "window_decode: alignment");
  if (need > 0 && (!workspace || workspace_bytes < need)) return fail(MV_ERR_WORKSPACE, "window_decode: workspace");
  WindowParams<__nv_bfloat16> p{};
  p.out = static_cast<__nv_bfloat16*>(out); p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_stride;
  p.cache = static_cast<const __nv_bfloat16*>(cache);
  p.tables = block_tables; p.bt_stride = bt_stride; p.max_blocks = max_blocks; p.block_size = block_size; p.num_blocks = num_blocks;
  p.positions = positions; p.bias = bias; p.bias_stride = bias_stride; p.distances = bias ? distances : 1;
  p.sink = static_cast<const __nv_bfloat16*>(sink); p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim;
  p.window = window; p.scale = scale; p.turn = reinterpret_cast<const float2*>(turn); p.table_rows = table_rows;
  p.splits = window_splits(batch, heads, kv_heads, std::max<int64_t>(most, 1));
  p.part_ml = static_cast<float*>(workspace);
  p.part_o = p.part_ml ? p.part_ml + static_cast<int64_t>(batch) * p.splits * heads * 2 : nullptr;
  auto st = static_cast<cudaStream_t>(stream);
  auto go = [&](auto kd) {
    constexpr int KD = decltype(kd)::value;
    if (vdim <= 64) return launch_window_decode<KD, 64>(p, batch, st);
    if (vdim <= 128) return launch_window_decode<KD, 128>(p, batch, st);
    return launch_window_decode<KD, 256>(p, batch, st);
  };
  if (dim <= 64) return go(std::integral_constant<int, 64>{});
  if (dim <= 128) return go(std::integral_constant<int, 128>{});
  return go(std::integral_constant<int, 256>{});
}

// ------------------------------------------------------------------------------------------------ two maps per head
static int64_t diff_most_keys(int64_t chunk, int max_blocks, int block_size) {
  return std::max<int64_t>(1, std::min<int64_t>(chunk, static_cast<int64_t>(max_blocks) * block_size));
}
// Bytes of scratch, or -1 when the kernel does not take the sizes.
extern "C" int64_t mv_diff_decode_workspace_bytes(int batch, int heads, int kv_heads, int dim, int vdim, int64_t most_keys) {
  using namespace mv;
  if (batch < 0 || batch > 65535 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || dim % 8 || vdim % 8 ||
      dim > 128 || vdim > 256 || most_keys <= 0)
    return -1;
  const int splits = window_splits(batch, heads, kv_heads, most_keys, 8);
  return splits == 1 ? 0 : static_cast<int64_t>(batch) * splits * heads * 2 * (vdim + 2) * 4;
}

extern "C" int mv_diff_decode(void* out, const void* q, int64_t q_stride, const void* cache, const int32_t* block_tables,
                              int64_t bt_stride, int max_blocks, int block_size, int64_t num_blocks,
                              const int64_t* positions, int64_t chunk, const void* gate, int64_t gate_stride, float lambda,
                              float mult, float eps, int batch, int heads, int kv_heads, int dim, int vdim, float scale,
                              void* workspace, int64_t workspace_bytes, void* stream) {
  using namespace mv;
  const int rc = check_window("diff_decode", heads, kv_heads, dim, vdim, chunk, block_size);
  if (rc) return rc;
  const int64_t most = diff_most_keys(chunk, max_blocks, block_size), need = mv_diff_decode_workspace_bytes(batch, heads, kv_heads, dim, vdim, most);
  if (need < 0) return fail(MV_ERR_LIMIT, "diff_decode: dim %d, vdim %d, batch %d", dim, vdim, batch);
  if (batch == 0) return MV_OK;
  if (!out || !q || !cache || !block_tables || !positions || !gate) return fail(MV_ERR_NULL, "diff_decode: null pointer");
  if (!aligned16(cache) || (reinterpret_cast<uintptr_t>(q) & 3u) || (reinterpret_cast<uintptr_t>(out) & 3u) || q_stride % 2)
    return fail(MV_ERR_ALIGN, "diff_decode: alignment");
  if (need > 0 && (!workspace || workspace_bytes < need)) return fail(MV_ERR_WORKSPACE, "diff_decode: workspace");
  WindowParams<__nv_bfloat16> p{};
  p.out = static_cast<__nv_bfloat16*>(out); p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_stride;
  p.cache = static_cast<const __nv_bfloat16*>(cache);
  p.tables = block_tables; p.bt_stride = bt_stride; p.max_blocks = max_blocks; p.block_size = block_size; p.num_blocks = num_blocks;
  p.positions = positions; p.distances = 1; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.scale = scale;
  p.window = 1LL << 40; p.maps = 2; p.chunk = chunk;
  p.gate = static_cast<const __nv_bfloat16*>(gate); p.gate_stride = gate_stride; p.lambda = lambda; p.mult = mult; p.eps = eps;
  p.splits = window_splits(batch, heads, kv_heads, most, 8);
  p.part_ml = static_cast<float*>(workspace);
  p.part_o = p.part_ml ? p.part_ml + static_cast<int64_t>(batch) * p.splits * heads * 4 : nullptr;
  auto st = static_cast<cudaStream_t>(stream);
  auto go = [&](auto kd) {
    constexpr int KD = decltype(kd)::value;
    if (vdim <= 64) return launch_window_decode<KD, 64, 2>(p, batch, st);
    if (vdim <= 128) return launch_window_decode<KD, 128, 2>(p, batch, st);
    return launch_window_decode<KD, 256, 2>(p, batch, st);
  };
  return dim <= 64 ? go(std::integral_constant<int, 64>{}) : go(std::integral_constant<int, 128>{});
}

extern "C" int mv_diff_norm_gate(void* out, const float* a, const void* gate, int64_t gate_stride, float lambda, float mult,
                                 float eps, int64_t tokens, int heads, int vdim, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "diff_norm_gate: dtype %d", dtype);
  if (tokens < 0 || heads <= 0 || vdim <= 0) return fail(MV_ERR_SHAPE, "diff_norm_gate: heads %d, vdim %d", heads, vdim);
  if (tokens == 0) return MV_OK;
  if (!out || !a || !gate) return fail(MV_ERR_NULL, "diff_norm_gate: null pointer");
  const unsigned grid = static_cast<unsigned>(std::min<int64_t>((tokens * heads + 7) / 8, kNumSMs * 32));
  auto run = [&](auto tag) {
    using T = decltype(tag);
    diff_norm_gate_kernel<T><<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(
        {static_cast<T*>(out), a, static_cast<const T*>(gate), gate_stride, tokens, heads, vdim, lambda, mult, eps});
    return check_launch("diff_norm_gate");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}
