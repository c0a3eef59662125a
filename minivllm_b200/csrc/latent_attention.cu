// Latent attention (keys and values are linear images of one low-rank row per token): preparation of a step's
// latent rows, and attention over the paged latent cache in its absorbed form, where the key up-projection has
// been moved to the query side, so that every head scores against the cached row [c | rotated key part] itself
// and returns a weighted sum of the c's.
//
// latent_prep_kernel: one CTA per token.  Normalises c, rotates the shared key part and every head's rotated
// query part, and scatters [c | k_rot] into the cache block the token's slot names.
// latent_attention_rows_kernel: any sizes, bf16 or fp32, any number of query rows per sequence.  fp32 arithmetic
// throughout.  It serves 32-bit models and sizes that the tensor-core kernels do not take.
#include "vec.cuh"

namespace mv {

constexpr int kLpThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kLpThreads)
latent_prep_kernel(T* __restrict__ q, int64_t q_stride, const T* __restrict__ down, int64_t down_stride,
                   const T* __restrict__ c_weight, const int64_t* __restrict__ positions,
                   const float* __restrict__ cos_t, const float* __restrict__ sin_t, int64_t max_position,
                   T* __restrict__ latent_out, T* __restrict__ cache, const int64_t* __restrict__ slot_mapping,
                   int64_t num_slots, int heads, int dim, int rot_dim, int rope_dims, int rank, float eps) {
  const int64_t t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int64_t pos = min(positions[t], max_position - 1);
  const int half = rope_dims / 2, row = rank + rot_dim;
  const float* ct = cos_t + pos * half;
  const float* st = sin_t + pos * half;
  const T* d = down + t * down_stride;
  T* lo = latent_out ? latent_out + t * row : nullptr;
  const int64_t slot = slot_mapping ? slot_mapping[t] : -1;
  T* co = cache && slot >= 0 && slot < num_slots ? cache + slot * row : nullptr;
  if (warp == 0) {
    float acc = 0.f;
    for (int i = lane; i < rank; i += 32) {
      const float v = Elem<T>::to_f(d[i]);
      acc = fmaf(v, v, acc);
    }
    const float rs = 1.f / sqrtf(warp_sum(acc) / static_cast<float>(rank) + eps);
    for (int i = lane; i < rank; i += 32) {
      const T v = Elem<T>::from_f(Elem<T>::to_f(d[i]) * rs * Elem<T>::to_f(c_weight[i]));
      if (lo) lo[i] = v;
      if (co) co[i] = v;
    }
  } else if (warp == 1) {
    for (int i = lane; i < rot_dim; i += 32) {
      float v = Elem<T>::to_f(d[rank + i]);
      if (i < half) v = v * ct[i] - Elem<T>::to_f(d[rank + i + half]) * st[i];
      else if (i < rope_dims) v = v * ct[i - half] + Elem<T>::to_f(d[rank + i - half]) * st[i - half];
      const T o = Elem<T>::from_f(v);
      if (lo) lo[rank + i] = o;
      if (co) co[rank + i] = o;
    }
  } else {
    T* qt = q + t * q_stride;
    for (int i = threadIdx.x - 64; i < heads * half; i += kLpThreads - 64) {
      const int h = i / half, j = i - h * half;
      T* r = qt + h * (dim + rot_dim) + dim;
      const float u = Elem<T>::to_f(r[j]), v = Elem<T>::to_f(r[j + half]);
      r[j] = Elem<T>::from_f(u * ct[j] - v * st[j]);
      r[j + half] = Elem<T>::from_f(v * ct[j] + u * st[j]);
    }
  }
}

// The same in 16-byte pieces: rank, dim and half of the rotated dimensions are multiples of 8 and rot_dim is rotated whole.
constexpr int kLvThreads = 128;
template <typename T>
__global__ void __launch_bounds__(kLvThreads)
latent_prep_vec_kernel(T* __restrict__ q, int64_t q_stride, const T* __restrict__ down, int64_t down_stride,
                       const T* __restrict__ c_weight, const int64_t* __restrict__ positions,
                       const float* __restrict__ cos_t, const float* __restrict__ sin_t, int64_t max_position,
                       T* __restrict__ latent_out, T* __restrict__ cache, const int64_t* __restrict__ slot_mapping,
                       int64_t num_slots, int heads, int dim, int rot_dim, int rank, float eps) {
  const int64_t t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int half = rot_dim / 2, row = rank + rot_dim, hv = half / 8;
  const T* d = down + t * down_stride;
  const int64_t slot = slot_mapping ? slot_mapping[t] : -1;
  T* lo = latent_out ? latent_out + t * row : nullptr;
  T* co = cache && slot >= 0 && slot < num_slots ? cache + slot * row : nullptr;
  if (warp == 0) {
    constexpr int kHold = 2;            // pieces of the row a lane keeps in registers (rank 512); longer rows re-read
    float hold[kHold][8];
    float acc = 0.f;
    for (int i = lane, k = 0; i < rank / 8; i += 32, ++k) {
      float v[8];
      Vec<T, 8>::load(d + i * 8, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc = fmaf(v[e], v[e], acc);
#pragma unroll
      for (int h = 0; h < kHold; ++h)
        if (k == h)
#pragma unroll
          for (int e = 0; e < 8; ++e) hold[h][e] = v[e];
    }
    const float rs = 1.f / sqrtf(warp_sum(acc) / static_cast<float>(rank) + eps);
    for (int i = lane, k = 0; i < rank / 8; i += 32, ++k) {
      float v[8], w[8];
      Vec<T, 8>::load(c_weight + i * 8, w);
      if (k >= kHold) Vec<T, 8>::load(d + i * 8, v);
#pragma unroll
      for (int h = 0; h < kHold; ++h)
        if (k == h)
#pragma unroll
          for (int e = 0; e < 8; ++e) v[e] = hold[h][e];
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = v[e] * rs * w[e];
      if (lo) Vec<T, 8>::store(lo + i * 8, v);
      if (co) Vec<T, 8>::store(co + i * 8, v);
    }
    return;
  }
  const int64_t pos = min(positions[t], max_position - 1);
  const float* ct = cos_t + pos * half;
  const float* st = sin_t + pos * half;
  // items: heads * hv pieces of the queries, then hv of the shared key part
  for (int i = threadIdx.x - 32; i < (heads + 1) * hv; i += kLvThreads - 32) {
    const int h = i / hv, j = (i - h * hv) * 8;
    const bool key = h == heads;
    const T* src = key ? d + rank : q + t * q_stride + static_cast<int64_t>(h) * (dim + rot_dim) + dim;
    float u[8], v[8], c[8], s[8];
    Vec<T, 8>::load(src + j, u);
    Vec<T, 8>::load(src + j + half, v);
    Vec<float, 8>::load(ct + j, c);
    Vec<float, 8>::load(st + j, s);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float a = u[e] * c[e] - v[e] * s[e];
      v[e] = v[e] * c[e] + u[e] * s[e];
      u[e] = a;
    }
    if (!key) {
      T* dst = q + t * q_stride + static_cast<int64_t>(h) * (dim + rot_dim) + dim;
      Vec<T, 8>::store(dst + j, u);
      Vec<T, 8>::store(dst + j + half, v);
    } else {
      if (lo) { Vec<T, 8>::store(lo + rank + j, u); Vec<T, 8>::store(lo + rank + j + half, v); }
      if (co) { Vec<T, 8>::store(co + rank + j, u); Vec<T, 8>::store(co + rank + j + half, v); }
    }
  }
}

constexpr int kLaThreads = 256;
constexpr int kLaHeads = 4;    // heads per CTA
constexpr int kLaKeys = 32;    // keys per tile
constexpr int kLaMaxRank = 1024, kLaMaxRow = 1536;
constexpr int kLaPer = kLaMaxRank / kLaThreads;

template <typename T>
__global__ void __launch_bounds__(kLaThreads)
latent_attention_rows_kernel(T* __restrict__ out, int64_t out_stride, int64_t out_head_stride,
                             const T* __restrict__ q_lat, int64_t q_lat_stride, int64_t q_lat_head_stride,
                             const T* __restrict__ q_rot, int64_t q_rot_stride, int64_t q_rot_head_stride,
                             const T* __restrict__ cache, const int32_t* __restrict__ block_tables, int64_t bt_stride,
                             int max_blocks, int block_size, int64_t num_blocks, const int32_t* __restrict__ cu_q,
                             int num_seqs, const int64_t* __restrict__ positions, const T* __restrict__ sink,
                             int heads, int rank, int rot_dim, float scale) {
  extern __shared__ __align__(16) float sm[];
  const int R = rank + rot_dim;
  float* sq = sm;                               // [kLaHeads][R]
  float* sk = sq + kLaHeads * R;                // [kLaKeys][R + 1]
  float* ss = sk + kLaKeys * (R + 1);           // [kLaHeads][kLaKeys]
  __shared__ float s_m[kLaHeads], s_l[kLaHeads], s_c[kLaHeads];
  const int t = blockIdx.x, h0 = blockIdx.y * kLaHeads, nh = min(kLaHeads, heads - h0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = seq_of_token(cu_q, num_seqs, t);
  const int32_t* table = block_tables + static_cast<int64_t>(seq) * bt_stride;
  const int64_t nk64 = min(positions[t] + 1, static_cast<int64_t>(max_blocks) * block_size);
  const int nk = static_cast<int>(nk64);
  for (int i = tid; i < kLaHeads * R; i += kLaThreads) {
    const int h = i / R, j = i - h * R;
    float v = 0.f;
    if (h < nh)
      v = j < rank ? Elem<T>::to_f(q_lat[t * q_lat_stride + (h0 + h) * q_lat_head_stride + j])
                   : Elem<T>::to_f(q_rot[t * q_rot_stride + (h0 + h) * q_rot_head_stride + j - rank]);
    sq[i] = v;
  }
  // the sink is one more score without a value: it opens the running maximum and sum
  if (tid < kLaHeads) {
    s_m[tid] = tid < nh && sink ? Elem<T>::to_f(sink[h0 + tid]) : -INFINITY;
    s_l[tid] = tid < nh && sink ? 1.f : 0.f;
  }
  float acc[kLaHeads][kLaPer];
#pragma unroll
  for (int h = 0; h < kLaHeads; ++h)
#pragma unroll
    for (int i = 0; i < kLaPer; ++i) acc[h][i] = 0.f;

  for (int k0 = 0; k0 < nk; k0 += kLaKeys) {
    __syncthreads();
    for (int k = warp; k < kLaKeys; k += kLaThreads / 32) {
      const int pos = k0 + k, blk = pos / block_size;
      const int32_t phys = pos < nk && blk < max_blocks ? table[blk] : -1;
      const bool ok = phys >= 0 && phys < num_blocks;
      const T* src = cache + (static_cast<int64_t>(ok ? phys : 0) * block_size + (pos - blk * block_size)) * R;
      for (int i = lane; i < R; i += 32) sk[k * (R + 1) + i] = ok ? Elem<T>::to_f(src[i]) : 0.f;
      if (lane < kLaHeads && !ok) ss[lane * kLaKeys + k] = -INFINITY;
      else if (lane < kLaHeads) ss[lane * kLaKeys + k] = 0.f;
    }
    __syncthreads();
    {  // two threads per (head, key)
      const int pair = tid >> 1, h = pair / kLaKeys, k = pair % kLaKeys, part = tid & 1;
      const float* a = sq + h * R;
      const float* b = sk + k * (R + 1);
      float s = 0.f;
      for (int i = part; i < R; i += 2) s = fmaf(a[i], b[i], s);
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      if (part == 0) ss[h * kLaKeys + k] += s * scale;     // -inf stays -inf
    }
    __syncthreads();
    if (warp < kLaHeads) {
      const float s = ss[warp * kLaKeys + lane];
      float mx = s;
#pragma unroll
      for (int o = 16; o; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_old = s_m[warp], m_new = fmaxf(m_old, mx);
      const float pr = m_new == -INFINITY ? 0.f : expf(s - m_new);
      const float sum = warp_sum(pr);
      ss[warp * kLaKeys + lane] = pr;
      if (lane == 0) {
        const float corr = m_new == -INFINITY ? 1.f : expf(m_old - m_new);
        s_c[warp] = corr;
        s_l[warp] = s_l[warp] * corr + sum;
        s_m[warp] = m_new;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kLaPer; ++i) {
      const int d = tid + i * kLaThreads;
      if (d < rank) {
#pragma unroll
        for (int h = 0; h < kLaHeads; ++h) acc[h][i] *= s_c[h];
        for (int k = 0; k < kLaKeys; ++k) {
          const float v = sk[k * (R + 1) + d];
#pragma unroll
          for (int h = 0; h < kLaHeads; ++h) acc[h][i] = fmaf(ss[h * kLaKeys + k], v, acc[h][i]);
        }
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int h = 0; h < kLaHeads; ++h) {
    if (h >= nh) break;
    const float l = s_l[h], inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
    for (int i = 0; i < kLaPer; ++i) {
      const int d = tid + i * kLaThreads;
      if (d < rank) out[t * out_stride + (h0 + h) * out_head_stride + d] = Elem<T>::from_f(acc[h][i] * inv);
    }
  }
}

}  // namespace mv

extern "C" int mv_latent_prep(void* q, int64_t q_stride, const void* down, int64_t down_stride, const void* c_weight,
                              const int64_t* positions, const float* cos_table, const float* sin_table,
                              int64_t max_position, void* latent_out, void* cache, const int64_t* slot_mapping,
                              int64_t num_slots, int64_t tokens, int heads, int dim, int rot_dim, int rope_dims,
                              int rank, float eps, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "latent_prep: dtype %d", dtype);
  if (tokens < 0 || heads <= 0 || dim < 0 || rot_dim < 0 || rank <= 0 || rope_dims % 2 || rope_dims > rot_dim || max_position <= 0)
    return fail(MV_ERR_SHAPE, "latent_prep: heads %d dim %d rot_dim %d rope %d rank %d", heads, dim, rot_dim, rope_dims, rank);
  if (tokens == 0) return MV_OK;
  if (!q || !down || !c_weight || !positions || !cos_table || !sin_table || (cache && !slot_mapping))
    return fail(MV_ERR_NULL, "latent_prep: null pointer");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int eb = sizeof(T);
    if (rank % 8 == 0 && dim % 8 == 0 && rot_dim % 16 == 0 && rope_dims == rot_dim && vec8_ok(q, q_stride, eb) &&
        vec8_ok(down, down_stride, eb) && aligned16(c_weight) && aligned16(cos_table) && aligned16(sin_table) &&
        aligned16(latent_out) && aligned16(cache)) {
      latent_prep_vec_kernel<T><<<static_cast<unsigned>(tokens), kLvThreads, 0, static_cast<cudaStream_t>(stream)>>>(
          static_cast<T*>(q), q_stride, static_cast<const T*>(down), down_stride, static_cast<const T*>(c_weight),
          positions, cos_table, sin_table, max_position, static_cast<T*>(latent_out), static_cast<T*>(cache),
          slot_mapping, num_slots, heads, dim, rot_dim, rank, eps);
      return check_launch("latent_prep");
    }
    latent_prep_kernel<T><<<static_cast<unsigned>(tokens), kLpThreads, 0, static_cast<cudaStream_t>(stream)>>>(
        static_cast<T*>(q), q_stride, static_cast<const T*>(down), down_stride, static_cast<const T*>(c_weight),
        positions, cos_table, sin_table, max_position, static_cast<T*>(latent_out), static_cast<T*>(cache),
        slot_mapping, num_slots, heads, dim, rot_dim, rope_dims, rank, eps);
    return check_launch("latent_prep");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_latent_attention_rows(void* out, int64_t out_stride, int64_t out_head_stride, const void* q_lat,
                                        int64_t q_lat_stride, int64_t q_lat_head_stride, const void* q_rot,
                                        int64_t q_rot_stride, int64_t q_rot_head_stride, const void* cache,
                                        const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size,
                                        int64_t num_blocks, const int32_t* cu_q, int num_seqs,
                                        const int64_t* positions, const void* sink, int64_t tokens, int heads,
                                        int rank, int rot_dim, float scale, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "latent_attention_rows: dtype %d", dtype);
  if (tokens < 0 || heads <= 0 || rank <= 0 || rot_dim < 0 || block_size <= 0 || max_blocks < 0)
    return fail(MV_ERR_SHAPE, "latent_attention_rows: heads %d rank %d rot_dim %d", heads, rank, rot_dim);
  if (rank > kLaMaxRank || rank + rot_dim > kLaMaxRow)
    return fail(MV_ERR_LIMIT, "latent_attention_rows: rank %d (at most %d), row %d (at most %d)", rank, kLaMaxRank, rank + rot_dim, kLaMaxRow);
  if (tokens == 0) return MV_OK;
  if (!out || !q_lat || (rot_dim && !q_rot) || !cache || !block_tables || !positions)
    return fail(MV_ERR_NULL, "latent_attention_rows: null pointer");
  const int R = rank + rot_dim;
  const size_t smem = sizeof(float) * (static_cast<size_t>(kLaHeads) * R + static_cast<size_t>(kLaKeys) * (R + 1) + kLaHeads * kLaKeys);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const cudaError_t e = cudaFuncSetAttribute(latent_attention_rows_kernel<T>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "latent_attention_rows: %s", cudaGetErrorString(e));
    const dim3 grid(static_cast<unsigned>(tokens), (heads + kLaHeads - 1) / kLaHeads);
    latent_attention_rows_kernel<T><<<grid, kLaThreads, smem, static_cast<cudaStream_t>(stream)>>>(
        static_cast<T*>(out), out_stride, out_head_stride, static_cast<const T*>(q_lat), q_lat_stride, q_lat_head_stride,
        static_cast<const T*>(q_rot), q_rot_stride,
        q_rot_head_stride, static_cast<const T*>(cache), block_tables, bt_stride, max_blocks, block_size, num_blocks,
        cu_q, num_seqs, positions, static_cast<const T*>(sink), heads, rank, rot_dim, scale);
    return check_launch("latent_attention_rows");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}
