// Rows of V consecutive elements as fp32 registers (V = 8 needs 16-byte aligned addresses, V = 1 none), and the
// few scalar functions the layers outside attention share.
#pragma once
#include "common.cuh"

namespace mv {

template <typename T, int V> struct Vec;
template <typename T> struct Vec<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&r)[1]) { r[0] = Elem<T>::to_f(*p); }
  static __device__ __forceinline__ void store(T* p, const float (&r)[1]) { *p = Elem<T>::from_f(r[0]); }
};
template <> struct Vec<float, 8> {
  static __device__ __forceinline__ void load(const float* p, float (&r)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    r[0] = a.x; r[1] = a.y; r[2] = a.z; r[3] = a.w; r[4] = b.x; r[5] = b.y; r[6] = b.z; r[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&r)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(r[0], r[1], r[2], r[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(r[4], r[5], r[6], r[7]);
  }
};
template <> struct Vec<__nv_bfloat16, 8> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&r)[8]) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      r[2 * i] = __uint_as_float(w[i] << 16);
      r[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&r)[8]) {
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 t = __floats2bfloat162_rn(r[2 * i], r[2 * i + 1]);
      w[i] = *reinterpret_cast<const uint32_t*>(&t);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  }
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
// Eight elements as they lie in memory, to be converted later (loads in flight cost no fp32 registers).
template <typename T> struct Raw8;
template <> struct Raw8<__nv_bfloat16> {
  uint4 v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void get(float (&r)[8]) const {
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      r[2 * i] = __uint_as_float(w[i] << 16);
      r[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  }
};
template <> struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) {
    a = *reinterpret_cast<const float4*>(p);
    b = *reinterpret_cast<const float4*>(p + 4);
  }
  __device__ __forceinline__ void get(float (&r)[8]) const {
    r[0] = a.x; r[1] = a.y; r[2] = a.z; r[3] = a.w; r[4] = b.x; r[5] = b.y; r[6] = b.z; r[7] = b.w;
  }
};

// Sigmoid and silu where the result is rounded to T: the special-function unit's exponential and reciprocal are far below the
// rounding of a 16-bit result.
template <typename T> __device__ __forceinline__ float sigmoid_t(float z) {
  return sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-z)) : sigmoid_f(z);
}
template <typename T> __device__ __forceinline__ float silu_t(float z) {
  return sizeof(T) == 2 ? __fdividef(z, 1.f + __expf(-z)) : silu_f(z);
}
// What a gate does to the value beside it (mv_act): output gates and the activations of gated feed-forwards.
template <typename T> __device__ __forceinline__ float glu_act(int act, float g, float u, float limit) {
  if (act == MV_ACT_SILU) return silu_t<T>(g) * u;
  if (act == MV_ACT_SIGMOID) return sigmoid_t<T>(g) * u;
  if (act == MV_ACT_GELU_TANH)       // 0.5 (1 + tanh(a)) = sigmoid(2 a)
    return g * sigmoid_t<T>(1.5957691216057308f * fmaf(0.044715f * g * g, g, g)) * u;
  if (act == MV_ACT_RELU) return fmaxf(g, 0.f) * u;
  g = fminf(g, limit);
  return g * sigmoid_t<T>(1.702f * g) * (fminf(fmaxf(u, -limit), limit) + 1.f);
}
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Sequence of token t in a packed batch: the s with cu[s] <= t < cu[s + 1].  cu == nullptr: one token each.
__device__ __forceinline__ int seq_of_token(const int32_t* cu, int num_seqs, int t) {
  if (cu == nullptr) return t;
  int lo = 0, hi = num_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// Host side: can rows at `p` with this element stride be read in chunks of eight?
inline bool vec8_ok(const void* p, int64_t stride_elems, int elem_bytes) {
  return p == nullptr || (aligned16(p) && (stride_elems * elem_bytes) % 16 == 0);
}

}  // namespace mv
