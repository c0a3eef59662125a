// Recurrences on a matrix state S (K x V, fp32) per sequence and head, read out once per token:
//   gated linear attention   S <- diag(alpha) S + k v^T,                             o = S^T q
//   gated delta rule         S <- g S;  u = beta (v - S^T k);  S <- S + k u^T,       o = S^T q
//   matrix memory (mLSTM)    S <- alpha S + w k v^T;  n <- alpha n + w k,            o = S^T q / (max(|n . q|, e^-m') + 1e-6)
//     with alpha = e^(f + m - m'), w = e^(i - m'), m' = max(f + m, i) the running maximum of the gates' logarithms
//   time mixing              o = (S + diag(u) k v^T)^T q,  S <- diag(e^(-e^z)) S + k v^T: the read-out comes before the decay,
//     and a token's own entry enters it with the bonus u
// Everything is computed in 32-bit, token by token, with the state in registers, so a result does not depend on how a
// prompt is cut.
//
// The columns of S are independent of one another.  A warp owns CW = VP * VT columns; a lane holds KT rows (in runs of
// four, interleaved over the KP lanes that share its columns) of VT columns, as packed pairs of rows, so that the
// products run as fma.rn.f32x2 and a float4 of k or q from shared memory serves two of them.  The sums over K meet in a
// reduce-scatter over the KP lanes: afterwards every lane holds one column's result.
//
// Decays near one enter as alpha - 1 (S + (alpha - 1) S): the rounding of alpha itself would add up over thousands of
// tokens.  For the same reason matrix memory forms f - (m' - m), which returns to S what the rounding of m' = f + m lost.
//
// The delta rule's scalar decay is kept out of the matrix: S = G * S', G the product of the decays, folded into S' when
// it becomes small.
//
// scan_kernel   prompts: one CTA per (sequence, head, block of value columns).  While a tile of tokens is worked on,
//               each warp has the next tile's token of its own in registers; it turns it into what the recurrence wants
//               (unit norms, decays, step sizes) in shared memory at the end of the tile.
//               Matrix memory: the chain of maxima comes from mlstm.cu; the first warp of the first block of columns keeps n
//               and leaves the denominators to the norm that follows.
// step_quad_kernel, step_kernel (vdim not a multiple of four)
//               one token per sequence: convolution (delta rule), one step of the state, the head's norm and the output
//               gate in one launch.  HBM-bound: 8 * heads * K * V bytes per sequence.
#pragma once
#include <algorithm>
#include <type_traits>
#include "vec.cuh"

namespace mv {

enum { SK_GLA = 0, SK_DELTA = 1, SK_MLSTM = 2, SK_TIME = 3 };

constexpr int log2_c(int n) { return n <= 1 ? 0 : 1 + log2_c(n / 2); }

template <int KIND_, int KP_, int KT_, int VT_> struct ScanShape {
  static constexpr int KIND = KIND_, KP = KP_, KT = KT_, VT = VT_;
  static constexpr int K = KP * KT;                       // padded rows
  static constexpr int VP = 32 / KP, CW = VP * VT;        // columns per warp
  static constexpr int NV = KIND == SK_DELTA ? 2 * VT : VT;              // sums per lane before the reduction
  static constexpr int SPLITS = log2_c(VT) < log2_c(KP) - (KIND == SK_DELTA) ? log2_c(VT) : log2_c(KP) - (KIND == SK_DELTA);
  static constexpr int HELD = VT >> SPLITS;               // columns per lane after it
  static constexpr int VBIT = KIND == SK_DELTA ? KP / 4 : KP / 2;        // lane bit of the first split of the columns
  static constexpr int LOW = VBIT >> (SPLITS ? SPLITS - 1 : 0);          // lanes that differ below it hold copies
  // lane (within the KP) that holds column v's sum
  static constexpr int holder(int v) {
    int l = 0;
    for (int i = 0; i < SPLITS; ++i)
      if ((v >> (log2_c(VT) - 1 - i)) & 1) l |= VBIT >> i;
    return l;
  }
  // first of the columns that lane kp holds
  static __device__ __forceinline__ int first_held(int kp) {
    int v = 0;
#pragma unroll
    for (int i = 0; i < SPLITS; ++i)
      if (kp & (VBIT >> i)) v |= VT >> (i + 1);
    return v;
  }
};

template <int N, int OFF> __device__ __forceinline__ void reduce_scatter(float* val, int kp) {
  if constexpr (OFF > 0) {
    if constexpr (N > 1) {
      const bool up = kp & OFF;
#pragma unroll
      for (int j = 0; j < N / 2; ++j) {
        const float send = up ? val[j] : val[j + N / 2], keep = up ? val[j + N / 2] : val[j];
        val[j] = keep + __shfl_xor_sync(0xffffffffu, send, OFF);
      }
      reduce_scatter<N / 2, OFF / 2>(val, kp);
    } else {
      val[0] += __shfl_xor_sync(0xffffffffu, val[0], OFF);
      reduce_scatter<1, OFF / 2>(val, kp);
    }
  }
}

// The rows and columns of one lane.
template <typename Sh> struct ScanState {
  float2 s[Sh::KT / 2][Sh::VT];
  float G;                        // delta rule: scale of s

  __device__ __forceinline__ void zero() {
    G = 1.f;
#pragma unroll
    for (int i = 0; i < Sh::KT / 2; ++i)
#pragma unroll
      for (int v = 0; v < Sh::VT; ++v) s[i][v] = make_float2(0.f, 0.f);
  }
  // src: column `col` of row 0 of the head's (K, V) state
  __device__ __forceinline__ void load(const float* src, int kp, int K, int V, int cols, bool vec) {
    G = 1.f;
#pragma unroll
    for (int i = 0; i < Sh::KT / 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (i * Sh::KP + kp) * 4 + e;
        float t[Sh::VT];
#pragma unroll
        for (int v = 0; v < Sh::VT; v += 4) {
          if (vec) {
            const float4 x = r < K && v < cols ? *reinterpret_cast<const float4*>(src + r * V + v) : make_float4(0.f, 0.f, 0.f, 0.f);
            t[v] = x.x; t[v + 1] = x.y; t[v + 2] = x.z; t[v + 3] = x.w;
          } else {
#pragma unroll
            for (int w = 0; w < 4; ++w) t[v + w] = r < K && v + w < cols ? src[r * V + v + w] : 0.f;
          }
        }
#pragma unroll
        for (int v = 0; v < Sh::VT; ++v) (e & 1 ? s[2 * i + e / 2][v].y : s[2 * i + e / 2][v].x) = t[v];
      }
  }
  __device__ __forceinline__ void store(float* dst, int kp, int K, int V, int cols, bool vec) const {
#pragma unroll
    for (int i = 0; i < Sh::KT / 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (i * Sh::KP + kp) * 4 + e;
        if (r >= K) continue;
#pragma unroll
        for (int v = 0; v < Sh::VT; v += 4) {
          float t[4];
#pragma unroll
          for (int w = 0; w < 4; ++w) t[w] = G * (e & 1 ? s[2 * i + e / 2][v + w].y : s[2 * i + e / 2][v + w].x);
          if (vec) {
            if (v < cols) *reinterpret_cast<float4*>(dst + r * V + v) = make_float4(t[0], t[1], t[2], t[3]);
          } else {
#pragma unroll
            for (int w = 0; w < 4; ++w)
              if (v + w < cols) dst[r * V + v + w] = t[w];
          }
        }
      }
  }
  // One token of gated linear attention.  sk, sq, sa: K values in shared memory (sa: alpha - 1); v: this lane's columns.
  // o receives the read-out of the columns first_held(kp) .. + HELD.  kBefore: of the state before the token.
  template <bool kBefore = false> __device__ __forceinline__ void gla(const float* sk, const float* sq, const float* sa, const float* sv, int kp, float (&o)[Sh::HELD]) {
    float2 acc[Sh::VT];
    float2 vv[Sh::VT];
#pragma unroll
    for (int v = 0; v < Sh::VT; v += 4) {
      const float4 x = *reinterpret_cast<const float4*>(sv + v);
      vv[v] = make_float2(x.x, x.x); vv[v + 1] = make_float2(x.y, x.y);
      vv[v + 2] = make_float2(x.z, x.z); vv[v + 3] = make_float2(x.w, x.w);
    }
#pragma unroll
    for (int v = 0; v < Sh::VT; ++v) acc[v] = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < Sh::KT / 4; ++i) {
      const float4 k4 = *reinterpret_cast<const float4*>(sk + (i * Sh::KP + kp) * 4);
      const float4 q4 = *reinterpret_cast<const float4*>(sq + (i * Sh::KP + kp) * 4);
      const float4 a4 = *reinterpret_cast<const float4*>(sa + (i * Sh::KP + kp) * 4);
#pragma unroll
      for (int v = 0; v < Sh::VT; ++v) {
        if (kBefore) {
          acc[v] = fma_f32x2(make_float2(q4.x, q4.y), s[2 * i][v], acc[v]);
          acc[v] = fma_f32x2(make_float2(q4.z, q4.w), s[2 * i + 1][v], acc[v]);
        }
        s[2 * i][v] = fma_f32x2(make_float2(k4.x, k4.y), vv[v], fma_f32x2(make_float2(a4.x, a4.y), s[2 * i][v], s[2 * i][v]));
        s[2 * i + 1][v] = fma_f32x2(make_float2(k4.z, k4.w), vv[v], fma_f32x2(make_float2(a4.z, a4.w), s[2 * i + 1][v], s[2 * i + 1][v]));
        if (!kBefore) {
          acc[v] = fma_f32x2(make_float2(q4.x, q4.y), s[2 * i][v], acc[v]);
          acc[v] = fma_f32x2(make_float2(q4.z, q4.w), s[2 * i + 1][v], acc[v]);
        }
      }
    }
    float val[Sh::VT];
#pragma unroll
    for (int v = 0; v < Sh::VT; ++v) val[v] = acc[v].x + acc[v].y;
    reduce_scatter<Sh::VT, Sh::KP / 2>(val, kp);
#pragma unroll
    for (int j = 0; j < Sh::HELD; ++j) o[j] = val[j];
  }
  // One token of the gated delta rule.  gm1: g - 1; ks, qs: factors of the stored k and q; kq: their product k . q, scaled.
  // Lanes with the bit KP / 2 of kp set receive the read-outs.
  __device__ __forceinline__ void delta(const float* sk, const float* sq, const float* sv, float gm1, float beta, float ks,
                                        float qs, float kq, int kp, float (&o)[Sh::HELD]) {
    float Gn = fmaf(G, gm1, G);
    if (Gn < 1e-6f) {
#pragma unroll
      for (int i = 0; i < Sh::KT / 2; ++i)
#pragma unroll
        for (int v = 0; v < Sh::VT; ++v) s[i][v] = mul_f32x2(s[i][v], make_float2(Gn, Gn));
      Gn = 1.f;
    }
    float4 k4[Sh::KT / 4];
    float2 ak[Sh::VT], aq[Sh::VT];
#pragma unroll
    for (int v = 0; v < Sh::VT; ++v) ak[v] = aq[v] = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < Sh::KT / 4; ++i) {
      k4[i] = *reinterpret_cast<const float4*>(sk + (i * Sh::KP + kp) * 4);
      const float4 q4 = *reinterpret_cast<const float4*>(sq + (i * Sh::KP + kp) * 4);
#pragma unroll
      for (int v = 0; v < Sh::VT; ++v) {
        ak[v] = fma_f32x2(make_float2(k4[i].x, k4[i].y), s[2 * i][v], ak[v]);
        ak[v] = fma_f32x2(make_float2(k4[i].z, k4[i].w), s[2 * i + 1][v], ak[v]);
        aq[v] = fma_f32x2(make_float2(q4.x, q4.y), s[2 * i][v], aq[v]);
        aq[v] = fma_f32x2(make_float2(q4.z, q4.w), s[2 * i + 1][v], aq[v]);
      }
    }
    float val[2 * Sh::VT];
#pragma unroll
    for (int v = 0; v < Sh::VT; ++v) {
      val[v] = ak[v].x + ak[v].y;
      val[Sh::VT + v] = aq[v].x + aq[v].y;
    }
    reduce_scatter<2 * Sh::VT, Sh::KP / 2>(val, kp);
    const float gk = Gn * ks, gq = Gn * qs, w = beta * ks / Gn;
    const int base = (threadIdx.x & 31) - kp, mine = Sh::first_held(kp);
#pragma unroll
    for (int j = 0; j < Sh::HELD; ++j) {
      const float dk = __shfl_xor_sync(0xffffffffu, val[j], Sh::KP / 2);     // S^T k of the columns this lane reads out
      o[j] = fmaf(gq, val[j], beta * fmaf(-gk, dk, sv[mine + j]) * kq);
    }
#pragma unroll
    for (int v = 0; v < Sh::VT; ++v) {
      const float dk = __shfl_sync(0xffffffffu, val[v & (Sh::HELD - 1)], base + Sh::holder(v));
      const float us = w * fmaf(-gk, dk, sv[v]);
      const float2 u2 = make_float2(us, us);
#pragma unroll
      for (int i = 0; i < Sh::KT / 4; ++i) {
        s[2 * i][v] = fma_f32x2(make_float2(k4[i].x, k4[i].y), u2, s[2 * i][v]);
        s[2 * i + 1][v] = fma_f32x2(make_float2(k4[i].z, k4[i].w), u2, s[2 * i + 1][v]);
      }
    }
    G = Gn;
  }
};

// Calls f with the shape for K rows.
template <int KIND, typename F> int scan_dispatch(int K, F&& f) {
  if (K <= 32) return f(ScanShape<KIND, 8, 4, 8>{});
  if (K <= 64) return f(ScanShape<KIND, 8, 8, 8>{});
  if (K <= 96) return f(ScanShape<KIND, 8, 12, 4>{});
  if (K <= 128) {
    if constexpr (KIND == SK_DELTA) return f(ScanShape<KIND, 8, 16, 4>{});
    else return f(ScanShape<KIND, 16, 8, 8>{});
  }
  return f(ScanShape<KIND, 16, 16, 4>{});
}
constexpr int kScanMaxK = 256;

// Logarithms of the decays, in 32-bit.
__device__ __forceinline__ float channel_log_decay(float z, float inv_tau) { return -softplus_f(-z) * inv_tau; }
// A decay below e^-40 is none that fp32 could tell from zero; sums of logarithms stay small enough for their differences.
__device__ __forceinline__ float time_log_decay(float z) { return -fminf(expf(z), 40.f); }
__device__ __forceinline__ float head_log_decay(float a, float A_log, float dt_bias) { return -expf(A_log) * softplus_f(a + dt_bias); }
constexpr float kUnitEps = 1e-6f;       // of q and k scaled to unit length
constexpr float kMemFloor = 1e-6f;      // matrix memory: added to the denominator

// Matrix memory: logarithms of the input and the forget gate from their logits.
__device__ __forceinline__ float mem_log_input(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float mem_log_forget(float z, float cap) { return -softplus_f(-cap * tanhf(z / cap)); }

constexpr int kScanMaxWarps = 8, kScanCols = 128;      // columns per CTA at most

template <typename T> struct ScanParams {
  T* out; int64_t out_stride;                          // (tokens, heads * V)
  const T *q, *k, *v; int64_t stride;                  // rows of a token: (kv_heads, K), (kv_heads, K), (heads, V)
  const T* z; int64_t z_stride;                        // gated linear attention: (heads, K) logits of the decay
  float inv_tau;
  const float* zf; int64_t zf_stride;                  // time mixing: (heads, K) logarithms of the decay's rate, to be added to w0
  const T *w0, *bonus;                                 //   (heads, K)
  const T *beta, *a; int64_t gate_stride;              // delta rule: (heads) logits of the step size and of the decay
  const T *A_log, *dt_bias;
  const float* gates; int64_t gates_stride;            // matrix memory, prompts: (heads) logits of the input gate, (heads) of the forget gate
  const T *x, *gates_w; int64_t x_stride; int width;   //   one token: (width) input of the gates, (2 heads, width) weights
  const T *i_b, *f_b; float cap;
  float *n_state, *m_state;                            //   (num_slots, heads, K), (num_slots, heads)
  const float4* chain; float* den;                     //   prompts: (tokens, heads) i, f, m, m' and denominators
  const int32_t *cu, *slots, *start;
  float* state; int num_slots, heads, kv_heads, K, V;
  float q_scale;
  // step only
  const T *gate, *norm_w; int64_t out_gate_stride; float eps, out_scale;
  const T *conv_w, *conv_state; int taps, channels;    // delta rule: channels [q | k | v]
};

template <typename Sh, typename T, int W>
__global__ void __launch_bounds__(32 * W, 16 / W) scan_kernel(const ScanParams<T> p, int cols_cta) {
  constexpr bool kDelta = Sh::KIND == SK_DELTA, kMem = Sh::KIND == SK_MLSTM, kTime = Sh::KIND == SK_TIME;
  constexpr int K = Sh::K, KL = K / 32, VL = kScanCols / 32, TT = W;      // a tile: one token per warp
  constexpr int VEC = kDelta ? 2 : 3;
  extern __shared__ __align__(16) float sm[];
  float* s_vec = sm;                                   // [2][TT][VEC][K]
  float* s_v = s_vec + 2 * TT * VEC * K;               // [2][TT][kScanCols]
  float* s_par = s_v + 2 * TT * kScanCols;             // [2][TT][4]: decay, step size, k . q; time mixing: k . (u q)
  const int s = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * cols_cta, pw = min(cols_cta, p.V - p0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kp = lane & (Sh::KP - 1), vp = lane / Sh::KP;
  const int kh = h / (p.heads / p.kv_heads);
  const int first = p.cu[s], n_tok = p.cu[s + 1] - first;
  if (n_tok <= 0) return;
  const int slot = p.slots[s], st0 = p.start[s];
  const bool live = slot >= 0 && slot < p.num_slots && st0 >= 0;
  const int c0 = warp * Sh::CW + vp * Sh::VT;          // this lane's first column within the block
  const bool work = warp * Sh::CW < pw, vec = p.V % 4 == 0;
  float* gS = p.state + (static_cast<int64_t>(live ? slot : 0) * p.heads + h) * p.K * p.V + p0 + c0;
  ScanState<Sh> S;
  if (work && live && st0 > 0) S.load(gS, kp, p.K, p.V, pw - c0, vec);
  else S.zero();

  T rk[KL], rq[KL], rv[VL], rb[2];
  std::conditional_t<kTime, float, T> rz[kDelta || kMem ? 1 : KL];
  float w0[kTime ? KL : 1], bonus[kTime ? KL : 1];
  if constexpr (kTime) {
#pragma unroll
    for (int m = 0; m < KL; ++m) {
      const bool ok = m * 32 + lane < p.K;
      w0[m] = ok ? Elem<T>::to_f(p.w0[h * p.K + m * 32 + lane]) : 0.f;
      bonus[m] = ok ? Elem<T>::to_f(p.bonus[h * p.K + m * 32 + lane]) : 0.f;
    }
  }
  float4 rc = make_float4(0.f, 0.f, 0.f, 0.f);
  float n[kMem ? KL : 1];                // matrix memory: this lane's entries of n
  const bool keeps_n = kMem && blockIdx.z == 0 && warp == 0;
  float* gN = kMem ? p.n_state + (static_cast<int64_t>(live ? slot : 0) * p.heads + h) * p.K : nullptr;
  if constexpr (kMem) {
#pragma unroll
    for (int m = 0; m < KL; ++m) n[m] = keeps_n && live && st0 > 0 && m * 32 + lane < p.K ? gN[m * 32 + lane] : 0.f;
  }
  float A_log = 0.f, dt_bias = 0.f;
  if (kDelta) {
    A_log = Elem<T>::to_f(p.A_log[h]);
    dt_bias = Elem<T>::to_f(p.dt_bias[h]);
  }
  const T zero_t = Elem<T>::from_f(0.f);
  auto fetch = [&](int t) {              // token `t` of the sequence into this warp's registers
    const bool on = t < n_tok;
    const int64_t row = first + t;
#pragma unroll
    for (int m = 0; m < KL; ++m) {
      const int j = m * 32 + lane;
      const bool ok = on && j < p.K;
      rk[m] = ok ? p.k[row * p.stride + kh * p.K + j] : zero_t;
      rq[m] = ok ? p.q[row * p.stride + kh * p.K + j] : zero_t;
      if constexpr (kTime) rz[m] = ok ? p.zf[row * p.zf_stride + h * p.K + j] : 0.f;
      else if constexpr (!kDelta && !kMem) rz[m] = ok ? p.z[row * p.z_stride + h * p.K + j] : zero_t;
    }
#pragma unroll
    for (int m = 0; m < VL; ++m) {
      const int j = m * 32 + lane;
      rv[m] = on && j < pw ? p.v[row * p.stride + static_cast<int64_t>(h) * p.V + p0 + j] : zero_t;
    }
    if (kMem && on) rc = p.chain[row * p.heads + h];
    if (kDelta) {
      rb[0] = on ? p.beta[row * p.gate_stride + h] : zero_t;
      rb[1] = on ? p.a[row * p.gate_stride + h] : zero_t;
    }
  };
  auto prepare = [&](int buf) {
    float* vecs = s_vec + (buf * TT + warp) * VEC * K;
    float kk = 0.f, qq = 0.f, kq = 0.f;
    const float alpha_m1 = kMem ? expm1f(rc.y - (rc.w - rc.z)) : 0.f, write = kMem ? expf(rc.x - rc.w) : 0.f;
    if (kMem && lane == 0) s_par[(buf * TT + warp) * 4] = expf(-rc.w);
#pragma unroll
    for (int m = 0; m < KL; ++m) {
      const int j = m * 32 + lane;
      const float kf = Elem<T>::to_f(rk[m]), qf = Elem<T>::to_f(rq[m]);
      if constexpr (kDelta) {
        kk = fmaf(kf, kf, kk);
        qq = fmaf(qf, qf, qq);
        kq = fmaf(kf, qf, kq);
        vecs[j] = kf;
        vecs[K + j] = qf;
      } else if constexpr (kMem) {
        vecs[j] = kf * write;
        vecs[K + j] = qf * p.q_scale;
        vecs[2 * K + j] = alpha_m1;
      } else if constexpr (kTime) {
        vecs[j] = kf;
        vecs[K + j] = qf;
        vecs[2 * K + j] = expm1f(time_log_decay(rz[m] + w0[m]));
        kq = fmaf(kf * bonus[m], qf, kq);
      } else {
        vecs[j] = kf;
        vecs[K + j] = qf * p.q_scale;
        vecs[2 * K + j] = expm1f(channel_log_decay(Elem<T>::to_f(rz[m]), p.inv_tau));
      }
    }
#pragma unroll
    for (int m = 0; m < VL; ++m) s_v[(buf * TT + warp) * kScanCols + m * 32 + lane] = Elem<T>::to_f(rv[m]);
    if (kTime) {
      kq = warp_sum(kq);
      if (lane == 0) s_par[(buf * TT + warp) * 4] = kq;
    }
    if (kDelta) {
      kk = warp_sum(kk);
      qq = warp_sum(qq);
      kq = warp_sum(kq);
      const float ks = 1.f / sqrtf(kk + kUnitEps), qs = p.q_scale / sqrtf(qq + kUnitEps);
#pragma unroll
      for (int m = 0; m < KL; ++m) {
        vecs[m * 32 + lane] *= ks;       // written by this lane above
        vecs[K + m * 32 + lane] *= qs;
      }
      if (lane == 0) {
        float* par = s_par + (buf * TT + warp) * 4;
        par[0] = expm1f(head_log_decay(Elem<T>::to_f(rb[1]), A_log, dt_bias));
        par[1] = sigmoid_f(Elem<T>::to_f(rb[0]));
        par[2] = kq * ks * qs;
      }
    }
  };
  fetch(warp);
  prepare(0);
  __syncthreads();
  T* out = p.out + static_cast<int64_t>(first) * p.out_stride + static_cast<int64_t>(h) * p.V + p0 + c0 + Sh::first_held(kp);
  const bool writes = work && (!kDelta || (kp & (Sh::KP / 2))) && (kp & (Sh::LOW - 1)) == 0;
  const int held = writes ? min(Sh::HELD, pw - c0 - Sh::first_held(kp)) : 0;
  for (int t0 = 0, buf = 0; t0 < n_tok; t0 += TT, buf ^= 1) {
    const bool more = t0 + TT < n_tok;
    if (more) fetch(t0 + TT + warp);
    if (work) {
      const int nt = min(TT, n_tok - t0);
      for (int t = 0; t < nt; ++t) {
        const float* vecs = s_vec + (buf * TT + t) * VEC * K;
        const float* sv = s_v + (buf * TT + t) * kScanCols + c0;
        float o[Sh::HELD];
        if constexpr (kDelta) {
          const float4 par = *reinterpret_cast<const float4*>(s_par + (buf * TT + t) * 4);
          S.delta(vecs, vecs + K, sv, par.x, par.y, 1.f, 1.f, par.z, kp, o);
        } else {
          S.template gla<kTime>(vecs, vecs + K, vecs + 2 * K, sv, kp, o);
        }
        if constexpr (kTime) {
          const float own = s_par[(buf * TT + t) * 4];
#pragma unroll
          for (int j = 0; j < Sh::HELD; ++j) o[j] = fmaf(own, sv[Sh::first_held(kp) + j], o[j]);
        }
#pragma unroll
        for (int j = 0; j < Sh::HELD; ++j)
          if (j < held) out[j] = Elem<T>::from_f(o[j]);
        out += p.out_stride;
        if constexpr (kMem) {
          if (!keeps_n) continue;
          float dot = 0.f;
#pragma unroll
          for (int m = 0; m < KL; ++m) {
            const int j = m * 32 + lane;
            n[m] = fmaf(vecs[2 * K], n[m], n[m]) + vecs[j];
            dot = fmaf(n[m], vecs[K + j], dot);
          }
          dot = warp_sum(dot);
          if (lane == 0)
            p.den[static_cast<int64_t>(first + t0 + t) * p.heads + h] = fmaxf(fabsf(dot), s_par[(buf * TT + t) * 4]) + kMemFloor;
        }
      }
    }
    if (more) prepare(buf ^ 1);
    __syncthreads();
  }
  if (live && work) S.store(gS, kp, p.K, p.V, pw - c0, vec);
  if constexpr (kMem) {
    if (keeps_n && live)
#pragma unroll
      for (int m = 0; m < KL; ++m)
        if (m * 32 + lane < p.K) gN[m * 32 + lane] = n[m];
  }
}

// Matrix memory: factors of the old state and of the new entry of a token, and its running maximum, for every thread of the
// block; the gates' logits are formed here.
struct MemFactors { float alpha_m1, write, m; };
template <typename T> __device__ __forceinline__ MemFactors mem_factors(const ScanParams<T>& p, int s, int h, int slot, int st0) {
  __shared__ float2 part[32];
  const T *x = p.x + static_cast<int64_t>(s) * p.x_stride, *wi = p.gates_w + static_cast<int64_t>(h) * p.width;
  const T* wf = wi + static_cast<int64_t>(p.heads) * p.width;
  float2 z = make_float2(0.f, 0.f);
  auto add = [&](float a, float bi, float bf) {
    z.x = fmaf(a, bi, z.x);
    z.y = fmaf(a, bf, z.y);
  };
  const uintptr_t bits = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(wi) | reinterpret_cast<uintptr_t>(wf);
  if ((bits & 15u) == 0 && p.width % 8 == 0) {
    for (int c = threadIdx.x * 8; c < p.width; c += blockDim.x * 8) {
      float a[8], bi[8], bf[8];
      Vec<T, 8>::load(x + c, a);
      Vec<T, 8>::load(wi + c, bi);
      Vec<T, 8>::load(wf + c, bf);
#pragma unroll
      for (int e = 0; e < 8; ++e) add(a[e], bi[e], bf[e]);
    }
  } else {
    for (int c = threadIdx.x; c < p.width; c += blockDim.x) add(Elem<T>::to_f(x[c]), Elem<T>::to_f(wi[c]), Elem<T>::to_f(wf[c]));
  }
  z = make_float2(warp_sum(z.x), warp_sum(z.y));
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = z;
  __syncthreads();
  z = make_float2(0.f, 0.f);
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) {
    z.x += part[w].x;
    z.y += part[w].y;
  }
  const float i = mem_log_input(z.x + Elem<T>::to_f(p.i_b[h]), p.cap), f = mem_log_forget(z.y + Elem<T>::to_f(p.f_b[h]), p.cap);
  const float old = st0 > 0 ? p.m_state[static_cast<int64_t>(slot) * p.heads + h] : 0.f;
  const float m = fmaxf(f + old, i);
  return {expm1f(f - (m - old)), expf(i - m), m};
}
// The state's n and m one token on, and the terms of n . q; between two barriers.
template <typename T>
__device__ __forceinline__ void mem_advance(const ScanParams<T>& p, int h, int slot, int st0, const MemFactors& f, const float* s_k,
                                            const float* s_q, float* s_nq) {
  float* gN = p.n_state + (static_cast<int64_t>(slot) * p.heads + h) * p.K;
  for (int j = threadIdx.x; j < p.K; j += blockDim.x) {
    const float old = st0 > 0 ? gN[j] : 0.f, n = fmaf(f.alpha_m1, old, old) + s_k[j];
    gN[j] = n;
    s_nq[j] = n * s_q[j];
  }
  if (threadIdx.x == 0) p.m_state[static_cast<int64_t>(slot) * p.heads + h] = f.m;
}

// The vectors of a token for the step kernels: K (padded) values of k and q, gated linear attention's alpha - 1, V (padded)
// values of v; the delta rule's go through the convolution, matrix memory's k takes its factor; time mixing: s_u = k times the bonus.
template <int KIND, typename T>
__device__ __forceinline__ void step_vectors(const ScanParams<T>& p, int s, int h, int slot, int st0, int K, int vpad, float* s_k,
                                             float* s_q, float* s_a, float* s_v, const MemFactors& mem, float* s_u) {
  constexpr bool kDelta = KIND == SK_DELTA, kMem = KIND == SK_MLSTM, kTime = KIND == SK_TIME;
  const int kh = h / (p.heads / p.kv_heads);
  for (int i = threadIdx.x; i < K + K + vpad; i += blockDim.x) {
    const int part = i < K ? 0 : i < 2 * K ? 1 : 2, j = part == 0 ? i : part == 1 ? i - K : i - 2 * K;
    const bool ok = j < (part == 2 ? p.V : p.K);
    float x = 0.f;
    if (ok) {
      const int c = part == 2 ? h * p.V + j : kh * p.K + j;
      const T* src = (part == 0 ? p.k : part == 1 ? p.q : p.v) + static_cast<int64_t>(s) * p.stride + c;
      x = Elem<T>::to_f(*src);
      if (kDelta) {
        const int ch = part == 0 ? p.kv_heads * p.K + c : part == 1 ? c : 2 * p.kv_heads * p.K + c;
        const T* wc = p.conv_w + static_cast<int64_t>(ch) * p.taps;
        const T* cs = p.conv_state + static_cast<int64_t>(slot) * (p.taps - 1) * p.channels + ch;
        float acc = 0.f;
        if (st0 > 0)
          for (int n = 0; n < p.taps - 1; ++n) acc = fmaf(Elem<T>::to_f(wc[n]), Elem<T>::to_f(cs[static_cast<int64_t>(n) * p.channels]), acc);
        acc = fmaf(Elem<T>::to_f(wc[p.taps - 1]), x, acc);
        x = Elem<T>::to_f(Elem<T>::from_f(silu_t<T>(acc)));       // rounded as the prompt path stores it
      } else if (part == 1 && !kTime) {
        x *= p.q_scale;
      } else if (kMem && part == 0) {
        x *= mem.write;
      }
    }
    (part == 0 ? s_k : part == 1 ? s_q : s_v)[j] = x;
    if (kMem && part == 0) s_a[j] = mem.alpha_m1;
    if (kTime && part == 0) s_u[j] = ok ? x * Elem<T>::to_f(p.bonus[h * p.K + j]) : 0.f;
    if (kTime && part == 0)
      s_a[j] = ok ? expm1f(time_log_decay(p.zf[static_cast<int64_t>(s) * p.zf_stride + h * p.K + j] + Elem<T>::to_f(p.w0[h * p.K + j]))) : 0.f;
    if (!kDelta && !kMem && !kTime && part == 0)
      s_a[j] = ok ? expm1f(channel_log_decay(Elem<T>::to_f(p.z[static_cast<int64_t>(s) * p.z_stride + h * p.K + j]), p.inv_tau)) : 0.f;
  }
}

// The delta rule's scalars of a token: g - 1, beta, the factors of k and q and their scaled product.  Every warp for itself.
struct StepFactors { float gm1, beta, ks, qs, kq; };
template <typename T>
__device__ __forceinline__ StepFactors step_factors(const ScanParams<T>& p, int s, int h, int K, const float* s_k, const float* s_q) {
  StepFactors f;
  const int64_t at = static_cast<int64_t>(s) * p.gate_stride + h;
  f.gm1 = expm1f(head_log_decay(Elem<T>::to_f(p.a[at]), Elem<T>::to_f(p.A_log[h]), Elem<T>::to_f(p.dt_bias[h])));
  f.beta = sigmoid_f(Elem<T>::to_f(p.beta[at]));
  float kk = 0.f, qq = 0.f, kq = 0.f;
  for (int j = threadIdx.x & 31; j < K; j += 32) {
    const float a = s_k[j], b = s_q[j];
    kk = fmaf(a, a, kk);
    qq = fmaf(b, b, qq);
    kq = fmaf(a, b, kq);
  }
  f.ks = 1.f / sqrtf(warp_sum(kk) + kUnitEps);
  f.qs = p.q_scale / sqrtf(warp_sum(qq) + kUnitEps);
  f.kq = warp_sum(kq) * f.ks * f.qs;
  return f;
}

// Time mixing: what a token's own entry adds to its read-out, per value.  Every warp for itself.
__device__ __forceinline__ float own_entry(int K, const float* s_u, const float* s_q) {
  float acc = 0.f;
  for (int j = threadIdx.x & 31; j < K; j += 32) acc = fmaf(s_u[j], s_q[j], acc);
  return warp_sum(acc);
}

template <typename T> __device__ __forceinline__ const T* step_gate(const ScanParams<T>& p, int s, int h) {
  return p.gate + static_cast<int64_t>(s) * p.out_gate_stride + static_cast<int64_t>(h) * p.V;
}
template <int KIND, typename T> __device__ __forceinline__ const T* step_weight(const ScanParams<T>& p, int h) {
  return p.norm_w + (KIND == SK_MLSTM || KIND == SK_TIME ? static_cast<int64_t>(h) * p.V : 0);
}
template <int KIND, typename T> __device__ __forceinline__ void step_ahead(const ScanParams<T>& p, int s, int h, T (&first)[2]) {
  const int j = threadIdx.x;
  first[0] = j < p.V ? step_gate<T>(p, s, h)[j] : Elem<T>::from_f(0.f);
  first[1] = j < p.V ? step_weight<KIND, T>(p, h)[j] : Elem<T>::from_f(0.f);
}
// Norm of the head's read-out and output gate; matrix memory divides first (s_nq: the terms of n . q).  `first`: gate and weight
// of this thread's first column, fetched ahead.
template <int KIND, typename T>
__device__ __forceinline__ void step_output(const ScanParams<T>& p, int s, int h, const float* s_o, T* out, const float* s_nq,
                                            const MemFactors& mem, const T (&first)[2]) {
  constexpr bool kMem = KIND == SK_MLSTM, kTime = KIND == SK_TIME;
  float inv = 1.f;
  if (kMem) {
    float dot = 0.f;
    for (int j = threadIdx.x & 31; j < p.K; j += 32) dot += s_nq[j];
    inv = 1.f / (fmaxf(fabsf(warp_sum(dot)), expf(-mem.m)) + kMemFloor);
  }
  float acc = 0.f;
  for (int j = threadIdx.x & 31; j < p.V; j += 32) acc = fmaf(s_o[j] * inv, s_o[j] * inv, acc);
  const float rs = inv / sqrtf(warp_sum(acc) / static_cast<float>(p.V) + p.eps);
  const T *gate = step_gate<T>(p, s, h), *w = step_weight<KIND, T>(p, h);
  for (int j = threadIdx.x; j < p.V; j += blockDim.x) {
    const bool ahead = j == static_cast<int>(threadIdx.x);
    const float g = Elem<T>::to_f(ahead ? first[0] : gate[j]), wj = Elem<T>::to_f(ahead ? first[1] : w[j]);
    out[j] = Elem<T>::from_f(s_o[j] * rs * wj * (kMem ? sigmoid_t<T>(g) : silu_t<T>(g)) * (kTime ? p.out_scale : 1.f));
  }
}

// Any sizes: the state in the prompt kernel's layout.
template <typename Sh, typename T>
__global__ void __launch_bounds__(256, 1) step_kernel(const ScanParams<T> p) {
  constexpr bool kDelta = Sh::KIND == SK_DELTA, kMem = Sh::KIND == SK_MLSTM, kTime = Sh::KIND == SK_TIME;
  constexpr int K = Sh::K;
  extern __shared__ __align__(16) float sm[];
  const int vpad = (p.V + Sh::CW - 1) / Sh::CW * Sh::CW;
  float *s_k = sm, *s_q = s_k + K, *s_a = s_q + K, *s_v = s_a + (kDelta ? 0 : K), *s_o = s_v + vpad, *s_nq = s_o + vpad;
  const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31, kp = lane & (Sh::KP - 1), vp = lane / Sh::KP, warps = blockDim.x >> 5;
  const int slot = p.slots[s], st0 = p.start[s];
  T* out = p.out + static_cast<int64_t>(s) * p.out_stride + static_cast<int64_t>(h) * p.V;
  if (slot < 0 || slot >= p.num_slots || st0 < 0) {
    for (int i = tid; i < p.V; i += blockDim.x) out[i] = Elem<T>::from_f(0.f);
    return;
  }
  const bool vec = p.V % 4 == 0;
  float* gS = p.state + (static_cast<int64_t>(slot) * p.heads + h) * p.K * p.V;
  T first[2];
  step_ahead<Sh::KIND>(p, s, h, first);
  MemFactors mem{};
  if constexpr (kMem) mem = mem_factors(p, s, h, slot, st0);
  step_vectors<Sh::KIND>(p, s, h, slot, st0, K, vpad, s_k, s_q, s_a, s_v, mem, s_nq);
  __syncthreads();
  if constexpr (kMem) mem_advance(p, h, slot, st0, mem, s_k, s_q, s_nq);
  StepFactors f{};
  if (kDelta) f = step_factors(p, s, h, K, s_k, s_q);
  const float own = kTime ? own_entry(p.K, s_nq, s_q) : 0.f;
  const bool writes = (!kDelta || (kp & (Sh::KP / 2))) && (kp & (Sh::LOW - 1)) == 0;
  ScanState<Sh> S;
  for (int cb = warp; cb * Sh::CW < p.V; cb += warps) {
    const int c0 = cb * Sh::CW + vp * Sh::VT;
    if (st0 > 0) S.load(gS + c0, kp, p.K, p.V, p.V - c0, vec);
    else S.zero();
    float o[Sh::HELD];
    if constexpr (kDelta) S.delta(s_k, s_q, s_v + c0, f.gm1, f.beta, f.ks, f.qs, f.kq, kp, o);
    else S.template gla<kTime>(s_k, s_q, s_a, s_v + c0, kp, o);
    if (writes)
#pragma unroll
      for (int j = 0; j < Sh::HELD; ++j) {
        const int c = c0 + Sh::first_held(kp) + j;
        s_o[c] = kTime ? fmaf(own, s_v[c], o[j]) : o[j];
      }
    S.store(gS + c0, kp, p.K, p.V, p.V - c0, vec);
  }
  __syncthreads();
  step_output<Sh::KIND>(p, s, h, s_o, out, s_nq, mem, first);
}

// vdim a multiple of four: a thread has four columns of every rows-th row of S, so that a warp reads whole lines, and the
// first kStHold of its rows in registers, requested before anything else.  The delta rule passes over S twice (read-outs,
// update); rows that are not held are read again, from L2.
constexpr int kStHold = 8, kStThreads4 = 512;
template <int KIND, typename T>
__global__ void __launch_bounds__(kStThreads4, 2) step_quad_kernel(const ScanParams<T> p, int vpad) {
  constexpr bool kDelta = KIND == SK_DELTA, kMem = KIND == SK_MLSTM, kTime = KIND == SK_TIME;
  extern __shared__ __align__(16) float sm[];
  const int K = (p.K + 3) & ~3, nthr = blockDim.x, tid = threadIdx.x, s = blockIdx.x, h = blockIdx.y;
  const int PQ = p.V / 4, rows = nthr / PQ, q = tid % PQ, r = tid / PQ;
  const bool on = r < rows;
  float *s_k = sm, *s_q = s_k + K, *s_a = s_q + K, *s_v = s_a + (kDelta ? 0 : K), *s_o = s_v + vpad;
  float* s_nq = s_o + vpad;                                      // matrix memory, time mixing
  float4* red = reinterpret_cast<float4*>(s_nq + (kMem || kTime ? K : 0));        // [rows][PQ], twice for the delta rule
  const int slot = p.slots[s], st0 = p.start[s];
  T* out = p.out + static_cast<int64_t>(s) * p.out_stride + static_cast<int64_t>(h) * p.V;
  if (slot < 0 || slot >= p.num_slots || st0 < 0) {
    for (int i = tid; i < p.V; i += nthr) out[i] = Elem<T>::from_f(0.f);
    return;
  }
  float4* gS = reinterpret_cast<float4*>(p.state + (static_cast<int64_t>(slot) * p.heads + h) * p.K * p.V) + q;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 x[kStHold];
  auto fetch = [&](int n0) {
#pragma unroll
    for (int i = 0; i < kStHold; ++i) {
      const int n = n0 + i * rows + r;
      x[i] = on && n < p.K && st0 > 0 ? gS[n * PQ] : zero;
    }
  };
  fetch(0);                              // in flight while the vectors are made
  T first[2];
  step_ahead<KIND>(p, s, h, first);
  MemFactors mem{};
  if constexpr (kMem) mem = mem_factors(p, s, h, slot, st0);
  step_vectors<KIND>(p, s, h, slot, st0, K, vpad, s_k, s_q, s_a, s_v, mem, s_nq);
  __syncthreads();
  if constexpr (kMem) mem_advance(p, h, slot, st0, mem, s_k, s_q, s_nq);
  const float4 v = on ? *reinterpret_cast<const float4*>(s_v + q * 4) : zero;
  float4 aq = zero, ak = zero;
  auto add = [](float w, const float4& y, float4& acc) {
    acc.x = fmaf(w, y.x, acc.x); acc.y = fmaf(w, y.y, acc.y); acc.z = fmaf(w, y.z, acc.z); acc.w = fmaf(w, y.w, acc.w);
  };
  const int span = kStHold * rows;
  if constexpr (!kDelta) {
    for (int n0 = 0; n0 < p.K; n0 += span) {
      if (n0) fetch(n0);
#pragma unroll
      for (int i = 0; i < kStHold; ++i) {
        const int n = n0 + i * rows + r;
        if (on && n < p.K) {
          const float a = s_a[n], k = s_k[n];
          const float4 old = x[i];
          if (kTime) add(s_q[n], old, aq);
          add(a, old, x[i]);
          add(k, v, x[i]);
          gS[n * PQ] = x[i];
          if (!kTime) add(s_q[n], x[i], aq);
        }
      }
    }
    if (on) red[r * PQ + q] = aq;
    const float own = kTime ? own_entry(p.K, s_nq, s_q) : 0.f;
    __syncthreads();
    for (int i = tid; i < p.V; i += nthr) {
      float o = kTime ? own * s_v[i] : 0.f;
      for (int k = 0; k < rows; ++k) o += reinterpret_cast<const float*>(red)[k * p.V + i];
      s_o[i] = o;
    }
  } else {
    const StepFactors f = step_factors(p, s, h, K, s_k, s_q);
    for (int n0 = 0; n0 < p.K; n0 += span) {
      if (n0 == 0) {
#pragma unroll
        for (int i = 0; i < kStHold; ++i) {
          const int n = i * rows + r;
          if (on && n < p.K) { add(s_k[n], x[i], ak); add(s_q[n], x[i], aq); }
        }
      } else {
#pragma unroll
        for (int i = 0; i < kStHold; ++i) {
          const int n = n0 + i * rows + r;
          if (on && n < p.K && st0 > 0) {
            const float4 y = gS[n * PQ];
            add(s_k[n], y, ak);
            add(s_q[n], y, aq);
          }
        }
      }
    }
    if (on) { red[r * PQ + q] = ak; red[(rows + r) * PQ + q] = aq; }
    __syncthreads();
    float4 u = zero;
    if (on) {
      float4 dk = zero;
      for (int k = 0; k < rows; ++k) add(1.f, red[k * PQ + q], dk);
      const float gk = (1.f + f.gm1) * f.ks;
      u = make_float4(f.beta * fmaf(-gk, dk.x, v.x), f.beta * fmaf(-gk, dk.y, v.y), f.beta * fmaf(-gk, dk.z, v.z), f.beta * fmaf(-gk, dk.w, v.w));
      if (r == 0) {
        float4 dq = zero;
        for (int k = 0; k < rows; ++k) add(1.f, red[(rows + k) * PQ + q], dq);
        const float gq = (1.f + f.gm1) * f.qs;
        *reinterpret_cast<float4*>(s_o + q * 4) = make_float4(fmaf(gq, dq.x, u.x * f.kq), fmaf(gq, dq.y, u.y * f.kq),
                                                              fmaf(gq, dq.z, u.z * f.kq), fmaf(gq, dq.w, u.w * f.kq));
      }
    }
    for (int n0 = 0; n0 < p.K; n0 += span) {
      if (n0) fetch(n0);
#pragma unroll
      for (int i = 0; i < kStHold; ++i) {
        const int n = n0 + i * rows + r;
        if (on && n < p.K) {
          const float4 old = x[i];
          add(f.gm1, old, x[i]);
          add(f.ks * s_k[n], u, x[i]);
          gS[n * PQ] = x[i];
        }
      }
    }
  }
  __syncthreads();
  step_output<KIND>(p, s, h, s_o, out, s_nq, mem, first);
}

template <typename Sh, typename T, int W>
static int launch_scan(const ScanParams<T>& p, int num_seqs, int cols, cudaStream_t st) {
  constexpr int VEC = Sh::KIND == SK_DELTA ? 2 : 3;
  const size_t smem = sizeof(float) * 2 * W * (VEC * Sh::K + kScanCols + 4);
  const cudaError_t e = cudaFuncSetAttribute(scan_kernel<Sh, T, W>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return fail(MV_ERR_CUDA, "state_scan: %s", cudaGetErrorString(e));
  scan_kernel<Sh, T, W><<<dim3(num_seqs, p.heads, (p.V + cols - 1) / cols), 32 * W, smem, st>>>(p, cols);
  return check_launch("state_scan");
}

template <int KIND, typename T> static int run_scan(const ScanParams<T>& p, int num_seqs, cudaStream_t st) {
  return scan_dispatch<KIND>(p.K, [&](auto sh) {
    using Sh = decltype(sh);
    // wide blocks share the preparation of a token among more columns; narrow ones fill the GPU when there is little work
    const int wide = std::min(kScanCols, kScanMaxWarps * Sh::CW), narrow = std::min(kScanCols, 4 * Sh::CW);
    const int64_t ctas = static_cast<int64_t>(num_seqs) * p.heads * ((p.V + wide - 1) / wide);
    if (wide > 4 * Sh::CW && p.V > narrow && ctas >= 2 * kNumSMs) return launch_scan<Sh, T, 8>(p, num_seqs, wide, st);
    return launch_scan<Sh, T, 4>(p, num_seqs, narrow, st);
  });
}

template <int KIND, typename T> static int run_step(const ScanParams<T>& p, int num_seqs, cudaStream_t st) {
  if (p.V % 4 == 0 && p.V <= 4 * kStThreads4) {
    const int quads = p.V / 4, K = (p.K + 3) & ~3;
    const int threads = std::min(kStThreads4, std::max(128, (quads * ((p.K + kStHold - 1) / kStHold) + 31) / 32 * 32));
    const int fit = std::max(threads, (quads + 31) / 32 * 32), rows = fit / quads;
    const size_t smem = sizeof(float) * ((KIND == SK_DELTA ? 2 : KIND == SK_GLA ? 3 : 4) * K + 2 * p.V + (KIND == SK_DELTA ? 2 : 1) * static_cast<size_t>(rows) * p.V);
    if (smem <= 48 * 1024) {
      step_quad_kernel<KIND, T><<<dim3(num_seqs, p.heads), fit, smem, st>>>(p, p.V);
      return check_launch("state_step");
    }
  }
  return scan_dispatch<KIND>(p.K, [&](auto sh) {
    using Sh = decltype(sh);
    const int blocks = (p.V + Sh::CW - 1) / Sh::CW, warps = std::min(8, blocks);
    const size_t smem = sizeof(float) * ((KIND == SK_DELTA ? 2 : KIND == SK_GLA ? 3 : 4) * Sh::K + 2 * static_cast<size_t>(blocks) * Sh::CW);
    if (smem > 48 * 1024) return fail(MV_ERR_LIMIT, "state_step: vdim %d", p.V);
    step_kernel<Sh, T><<<dim3(num_seqs, p.heads), 32 * warps, smem, st>>>(p);
    return check_launch("state_step");
  });
}

static int check_scan(const char* what, int dtype, int num_seqs, int heads, int kv_heads, int K, int V) {
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "%s: dtype %d", what, dtype);
  if (num_seqs < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || K <= 0 || V <= 0)
    return fail(MV_ERR_SHAPE, "%s: heads %d over %d, dim %d, vdim %d", what, heads, kv_heads, K, V);
  if (K > kScanMaxK) return fail(MV_ERR_LIMIT, "%s: dim %d (at most %d)", what, K, kScanMaxK);
  if (heads > 65535) return fail(MV_ERR_LIMIT, "%s: %d heads", what, heads);
  return MV_OK;
}

}  // namespace mv
