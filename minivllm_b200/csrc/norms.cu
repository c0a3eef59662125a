// What stands between two sublayers of a decoder whose residual stream is fp32 and whose RMS norms work on
// groups of channels: one launch takes a sublayer's result (or the embedding row, or the pieces of a mixture of
// experts), gates it element by element, normalises it, adds it to the residual stream, normalises the sum and
// writes the next sublayer's input.  Plus the gated group norm that ends a state-space mixer, and a sigmoid gate.
//
// HBM-bound.  A CTA owns a row and keeps it in shared memory as fp32; every group of channels belongs to a fixed
// set of warps, so sums are formed in a fixed order whatever the batch.
#include <algorithm>
#include <type_traits>
#include "vec.cuh"

namespace mv {

constexpr int kNormThreads = 256;
constexpr int kNormWarps = kNormThreads / 32;
constexpr int kMaxTop = 256;     // choices per token

enum { SRC_EMBED = 0, SRC_ROWS = 1, SRC_EXPERTS = 2, SRC_PAIR = 3 };

template <typename T> struct ResidualParams {
  T* out;                  // (rows, width): normalised residual, or the residual itself without w_next
  float* x;                // (rows, width): residual stream, updated (SRC_EMBED: written)
  const T* y; int64_t y_stride;                 // SRC_ROWS: sublayer result;  SRC_EXPERTS: expert rows (sorted)
  const T* gate; int64_t gate_stride; const T* gate_bias;   // logits of the element gate (null: no gate)
  const T* y2; int64_t y2_stride; const T* w_y; const T* w_y2;   // SRC_PAIR: half the sum of norm(y) w_y and norm(y2) w_y2
  const T* w_post;         // norm of the sublayer's result (SRC_EMBED: of the embedding row, may be null)
  const T* w_next;         // norm of the new residual (null: none)
  const int64_t* ids; const T* embed; int64_t vocab;        // SRC_EMBED
  const int32_t* pos; const float* topw; int top;           // SRC_EXPERTS: row of (token, k) and its weight
  const T* shared; int64_t shared_stride; const T* sg; int64_t sg_stride;   // shared expert and its scalar gate
  float mult;
  int width, groups;
  float eps;
};

// Which warps sum which group: `wpg` warps each, `cg` groups at a time.
struct GroupPlan {
  int wpg, cg, g0, sub, chunks, gs;
  __device__ __forceinline__ GroupPlan(int width, int groups, int V, int warp) {
    wpg = groups >= kNormWarps ? 1 : kNormWarps / groups;
    cg = kNormWarps / wpg;
    g0 = warp / wpg;
    sub = warp - g0 * wpg;
    gs = width / groups;
    chunks = gs / V;
    if (g0 >= cg) g0 = groups;   // left-over warps
  }
};
__device__ __forceinline__ float group_rs(const float* part, int g, int wpg, int gs, float eps) {
  float s = 0.f;
  for (int k = 0; k < wpg; ++k) s += part[g * wpg + k];
  return 1.f / sqrtf(s / static_cast<float>(gs) + eps);
}

template <typename T, int V, int SRC>
__global__ void __launch_bounds__(kNormThreads) residual_norm_kernel(const ResidualParams<T> p) {
  extern __shared__ __align__(16) float s_row[];
  float* part = s_row + ((p.width + 3) & ~3);
  float* part2 = part + (p.groups < kNormWarps ? kNormWarps : p.groups);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int64_t row = blockIdx.x;
  const GroupPlan gp(p.width, p.groups, V, warp);
  const bool post = SRC != SRC_EMBED || p.w_post;
  float* x = p.x + row * p.width;
  float sgate = 0.f;
  if (SRC == SRC_PAIR) {       // sums of squares of both rows
    for (int g = gp.g0; g < p.groups; g += gp.cg) {
      float a = 0.f, b = 0.f;
      for (int i = gp.sub * 32 + lane; i < gp.chunks; i += gp.wpg * 32) {
        const int c = g * gp.gs + i * V;
        float u[V], v[V];
        Vec<T, V>::load(p.y + row * p.y_stride + c, u);
        Vec<T, V>::load(p.y2 + row * p.y2_stride + c, v);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          a = fmaf(u[e], u[e], a);
          b = fmaf(v[e], v[e], b);
        }
      }
      a = warp_sum(a);
      b = warp_sum(b);
      if (lane == 0) {
        part[g * gp.wpg + gp.sub] = a;
        part2[g * gp.wpg + gp.sub] = b;
      }
    }
    __syncthreads();
    for (int g = gp.g0; g < p.groups; g += gp.cg) {
      const float ra = 0.5f * group_rs(part, g, gp.wpg, gp.gs, p.eps), rb = 0.5f * group_rs(part2, g, gp.wpg, gp.gs, p.eps);
      for (int i = gp.sub * 32 + lane; i < gp.chunks; i += gp.wpg * 32) {
        const int c = g * gp.gs + i * V;
        float u[V], v[V], wu[V], wv[V];
        Vec<T, V>::load(p.y + row * p.y_stride + c, u);
        Vec<T, V>::load(p.y2 + row * p.y2_stride + c, v);
        Vec<T, V>::load(p.w_y + c, wu);
        Vec<T, V>::load(p.w_y2 + c, wv);
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = u[e] * ra * wu[e] + v[e] * rb * wv[e];
        Vec<float, V>::store(s_row + c, u);      // read back by the thread that wrote it
      }
    }
    __syncthreads();
  }
  int64_t token = 0;
  if (SRC == SRC_EMBED) {
    token = p.ids[row];
    if (token < 0 || token >= p.vocab) token = 0;   // placeholder rows of a padded batch
  }
  __shared__ int s_pos[SRC == SRC_EXPERTS ? kMaxTop : 1];
  __shared__ float s_w[SRC == SRC_EXPERTS ? kMaxTop : 1];
  if (SRC == SRC_EXPERTS) {
    for (int k = threadIdx.x; k < p.top; k += kNormThreads) {
      s_pos[k] = p.pos[row * p.top + k];
      s_w[k] = p.topw[row * p.top + k];
    }
    __syncthreads();
  }
  if (SRC == SRC_EXPERTS && p.shared) sgate = p.sg ? sigmoid_f(Elem<T>::to_f(p.sg[row * p.sg_stride])) : 1.f;

  for (int g = gp.g0; g < p.groups; g += gp.cg) {
    float acc = 0.f;
    for (int i = gp.sub * 32 + lane; i < gp.chunks; i += gp.wpg * 32) {
      const int c = g * gp.gs + i * V;
      float v[V];
      if (SRC == SRC_EMBED) {
        Vec<T, V>::load(p.embed + token * p.width + c, v);
        if (!post) Vec<float, V>::store(x + c, v);
      } else {
        if (SRC == SRC_ROWS) {
          Vec<T, V>::load(p.y + row * p.y_stride + c, v);
        } else if (SRC == SRC_PAIR) {
          Vec<float, V>::load(s_row + c, v);
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e) v[e] = 0.f;
          constexpr int kAtOnce = 4;
          for (int k0 = 0; k0 < p.top; k0 += kAtOnce) {
            float t[kAtOnce][V];
#pragma unroll
            for (int k = 0; k < kAtOnce; ++k)
              if (k0 + k < p.top) Vec<T, V>::load(p.y + static_cast<int64_t>(s_pos[k0 + k]) * p.y_stride + c, t[k]);
#pragma unroll
            for (int k = 0; k < kAtOnce; ++k)
              if (k0 + k < p.top) {
#pragma unroll
                for (int e = 0; e < V; ++e) v[e] = fmaf(s_w[k0 + k], t[k][e], v[e]);
              }
          }
          if (p.shared) {
            float t[V];
            Vec<T, V>::load(p.shared + row * p.shared_stride + c, t);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = fmaf(sgate, t[e], v[e]);
          }
        }
        if (p.gate) {
          float t[V], b[V];
          Vec<T, V>::load(p.gate + row * p.gate_stride + c, t);
          Vec<T, V>::load(p.gate_bias + c, b);
#pragma unroll
          for (int e = 0; e < V; ++e) v[e] *= sigmoid_t<T>(t[e] + b[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) acc = fmaf(v[e], v[e], acc);
      Vec<float, V>::store(s_row + c, v);
    }
    acc = warp_sum(acc);
    if (lane == 0) part[g * gp.wpg + gp.sub] = acc;
  }
  __syncthreads();
  const float* fin = part;
  if (post) {
    for (int g = gp.g0; g < p.groups; g += gp.cg) {
      const float rs = group_rs(part, g, gp.wpg, gp.gs, p.eps);
      float acc = 0.f;
      for (int i = gp.sub * 32 + lane; i < gp.chunks; i += gp.wpg * 32) {
        const int c = g * gp.gs + i * V;
        float v[V], w[V], r[V];
        Vec<float, V>::load(s_row + c, v);
        Vec<T, V>::load(p.w_post + c, w);
        if (SRC != SRC_EMBED) Vec<float, V>::load(x + c, r);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          r[e] = SRC == SRC_EMBED ? v[e] * rs * w[e] : fmaf(p.mult, v[e] * rs * w[e], r[e]);
          acc = fmaf(r[e], r[e], acc);
        }
        Vec<float, V>::store(x + c, r);
        Vec<float, V>::store(s_row + c, r);
      }
      acc = warp_sum(acc);
      if (lane == 0) part2[g * gp.wpg + gp.sub] = acc;
    }
    __syncthreads();
    fin = part2;
  }
  for (int g = gp.g0; g < p.groups; g += gp.cg) {
    const float rs = group_rs(fin, g, gp.wpg, gp.gs, p.eps);
    for (int i = gp.sub * 32 + lane; i < gp.chunks; i += gp.wpg * 32) {
      const int c = g * gp.gs + i * V;
      float v[V], w[V];
      Vec<float, V>::load(s_row + c, v);
      if (p.w_next) {
        Vec<T, V>::load(p.w_next + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = v[e] * rs * w[e];
      }
      Vec<T, V>::store(p.out + row * p.width + c, v);
    }
  }
}

// The same with the row in registers: at most eight groups, kCh pieces of eight channels per thread.  Everything a row
// needs is requested at once; two block-wide sums follow.
template <typename T, int SRC, int kCh>
__global__ void __launch_bounds__(kNormThreads, SRC == SRC_EXPERTS ? (kCh == 1 ? 3 : 2) : SRC == SRC_PAIR && kCh == 2 ? 2 : 3) residual_norm_reg_kernel(const ResidualParams<T> p) {
  __shared__ float part[kNormWarps], part2[kNormWarps], part3[SRC == SRC_PAIR ? 2 * kNormWarps : 1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int64_t row = blockIdx.x;
  const GroupPlan gp(p.width, p.groups, 8, warp);
  const bool on = gp.g0 < p.groups, post = SRC != SRC_EMBED || p.w_post;
  float* x = p.x + row * p.width;
  int col[kCh];
  bool has[kCh];
#pragma unroll
  for (int k = 0; k < kCh; ++k) {
    const int i = gp.sub * 32 + lane + k * gp.wpg * 32;
    has[k] = on && i < gp.chunks;
    col[k] = gp.g0 * gp.gs + i * 8;
  }
  float v[kCh][8], r[kCh][8];
  Raw8<T> gate[kCh], gb[kCh], wp[kCh], wn[kCh];
  int64_t token = 0;
  float sgate = 0.f;
  if (SRC == SRC_EMBED) {
    token = p.ids[row];
    if (token < 0 || token >= p.vocab) token = 0;
  }
  if (SRC == SRC_EXPERTS && p.shared) sgate = p.sg ? sigmoid_f(Elem<T>::to_f(p.sg[row * p.sg_stride])) : 1.f;
#pragma unroll
  for (int k = 0; k < kCh; ++k)
    if (has[k]) {
      if (p.w_next) wn[k].load(p.w_next + col[k]);
      if (post) wp[k].load(p.w_post + col[k]);
      if (SRC != SRC_EMBED) {
        Vec<float, 8>::load(x + col[k], r[k]);
        if (p.gate) {
          gate[k].load(p.gate + row * p.gate_stride + col[k]);
          gb[k].load(p.gate_bias + col[k]);
        }
      }
    }
  if (SRC == SRC_EXPERTS) {
    Raw8<T> sh[kCh];
#pragma unroll
    for (int k = 0; k < kCh; ++k) {
      if (has[k] && p.shared) sh[k].load(p.shared + row * p.shared_stride + col[k]);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[k][e] = 0.f;
    }
    constexpr int kAtOnce = kCh == 1 ? 6 : 4;
    for (int k0 = 0; k0 < p.top; k0 += kAtOnce) {
      int64_t at[kAtOnce];
      float w[kAtOnce];
#pragma unroll
      for (int j = 0; j < kAtOnce; ++j) {
        const bool ok = k0 + j < p.top;
        at[j] = ok ? static_cast<int64_t>(p.pos[row * p.top + k0 + j]) * p.y_stride : 0;
        w[j] = ok ? p.topw[row * p.top + k0 + j] : 0.f;
      }
#pragma unroll
      for (int k = 0; k < kCh; ++k)
        if (has[k]) {
          Raw8<T> t[kAtOnce];
#pragma unroll
          for (int j = 0; j < kAtOnce; ++j)
            if (k0 + j < p.top) t[j].load(p.y + at[j] + col[k]);
#pragma unroll
          for (int j = 0; j < kAtOnce; ++j)
            if (k0 + j < p.top) {
              float f[8];
              t[j].get(f);
#pragma unroll
              for (int e = 0; e < 8; ++e) v[k][e] = fmaf(w[j], f[e], v[k][e]);
            }
        }
    }
#pragma unroll
    for (int k = 0; k < kCh; ++k)
      if (has[k] && p.shared) {
        float f[8];
        sh[k].get(f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[k][e] = fmaf(sgate, f[e], v[k][e]);
      }
  } else if (SRC == SRC_PAIR) {
    Raw8<T> a[kCh], b[kCh], wa[kCh], wb[kCh];
#pragma unroll
    for (int k = 0; k < kCh; ++k)
      if (has[k]) {
        a[k].load(p.y + row * p.y_stride + col[k]);
        b[k].load(p.y2 + row * p.y2_stride + col[k]);
        wa[k].load(p.w_y + col[k]);
        wb[k].load(p.w_y2 + col[k]);
      }
    float sa = 0.f, sb = 0.f;
#pragma unroll
    for (int k = 0; k < kCh; ++k)
      if (has[k]) {
        float u[8], t[8];
        a[k].get(u);
        b[k].get(t);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          sa = fmaf(u[e], u[e], sa);
          sb = fmaf(t[e], t[e], sb);
        }
      }
    sa = warp_sum(sa);
    sb = warp_sum(sb);
    if (lane == 0) {
      part3[warp] = sa;
      part3[kNormWarps + warp] = sb;
    }
    __syncthreads();
    const float ra = on ? 0.5f * group_rs(part3, gp.g0, gp.wpg, gp.gs, p.eps) : 0.f;
    const float rb = on ? 0.5f * group_rs(part3 + kNormWarps, gp.g0, gp.wpg, gp.gs, p.eps) : 0.f;
#pragma unroll
    for (int k = 0; k < kCh; ++k)
      if (has[k]) {
        float u[8], t[8], wu[8], wt[8];
        a[k].get(u);
        b[k].get(t);
        wa[k].get(wu);
        wb[k].get(wt);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[k][e] = u[e] * ra * wu[e] + t[e] * rb * wt[e];
      }
  } else {
#pragma unroll
    for (int k = 0; k < kCh; ++k)
      if (has[k]) Vec<T, 8>::load(SRC == SRC_EMBED ? p.embed + token * p.width + col[k] : p.y + row * p.y_stride + col[k], v[k]);
  }
  float acc = 0.f;
#pragma unroll
  for (int k = 0; k < kCh; ++k)
    if (has[k]) {
      if (!post) Vec<float, 8>::store(x + col[k], v[k]);
      if (SRC != SRC_EMBED && p.gate) {
        float t[8], b[8];
        gate[k].get(t);
        gb[k].get(b);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[k][e] *= sigmoid_t<T>(t[e] + b[e]);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) acc = fmaf(v[k][e], v[k][e], acc);
    }
  acc = warp_sum(acc);
  if (lane == 0) part[warp] = acc;
  __syncthreads();
  const float* fin = part;
  if (post) {
    const float rs = on ? group_rs(part, gp.g0, gp.wpg, gp.gs, p.eps) : 0.f;
    acc = 0.f;
#pragma unroll
    for (int k = 0; k < kCh; ++k)
      if (has[k]) {
        float w[8];
        wp[k].get(w);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          v[k][e] = SRC == SRC_EMBED ? v[k][e] * rs * w[e] : fmaf(p.mult, v[k][e] * rs * w[e], r[k][e]);
          acc = fmaf(v[k][e], v[k][e], acc);
        }
        Vec<float, 8>::store(x + col[k], v[k]);
      }
    acc = warp_sum(acc);
    if (lane == 0) part2[warp] = acc;
    __syncthreads();
    fin = part2;
  }
  const float rs = on ? group_rs(fin, gp.g0, gp.wpg, gp.gs, p.eps) : 0.f;
#pragma unroll
  for (int k = 0; k < kCh; ++k)
    if (has[k]) {
      if (p.w_next) {
        float w[8];
        wn[k].get(w);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[k][e] = v[k][e] * rs * w[e];
      }
      Vec<T, 8>::store(p.out + row * p.width + col[k], v[k]);
    }
}

// What follows a norm per head: the read-outs' denominators (rows, heads), null: none; the norm's weight for the whole row
// instead of one that the heads share; the gate's activation.
struct HeadNorm {
  const float* den;
  bool full_weight, sigmoid;
  float mult;                    // of the result
  int64_t out_stride;            // of its rows, 0: dense
};

// kGateFirst: out = group_rms_norm(y * silu(z)) * w.  Otherwise out = group_rms_norm(y / den) * w * act(z).
template <typename T, int V, bool kGateFirst>
__global__ void __launch_bounds__(kNormThreads)
gated_group_norm_kernel(T* __restrict__ out, const T* __restrict__ y, int64_t y_stride, const T* __restrict__ z,
                        int64_t z_stride, const T* __restrict__ w, int width, int groups, float eps, const HeadNorm hn) {
  extern __shared__ __align__(16) float s_row[];
  float* part = s_row + ((width + 3) & ~3);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int64_t row = blockIdx.x;
  const GroupPlan gp(width, groups, V, warp);
  for (int g = gp.g0; g < groups; g += gp.cg) {
    float acc = 0.f;
    const float den = !kGateFirst && hn.den ? 1.f / hn.den[row * groups + g] : 1.f;
    for (int i = gp.sub * 32 + lane; i < gp.chunks; i += gp.wpg * 32) {
      const int c = g * gp.gs + i * V;
      float v[V], t[V];
      Vec<T, V>::load(y + row * y_stride + c, v);
      if (kGateFirst) Vec<T, V>::load(z + row * z_stride + c, t);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        v[e] *= kGateFirst ? silu_t<T>(t[e]) : den;
        acc = fmaf(v[e], v[e], acc);
      }
      Vec<float, V>::store(s_row + c, v);
    }
    acc = warp_sum(acc);
    if (lane == 0) part[g * gp.wpg + gp.sub] = acc;
  }
  __syncthreads();
  for (int g = gp.g0; g < groups; g += gp.cg) {
    const float rs = group_rs(part, g, gp.wpg, gp.gs, eps);
    for (int i = gp.sub * 32 + lane; i < gp.chunks; i += gp.wpg * 32) {
      const int c = g * gp.gs + i * V;
      float v[V], t[V];
      Vec<float, V>::load(s_row + c, v);
      Vec<T, V>::load(w + (kGateFirst || hn.full_weight ? c : c - g * gp.gs), t);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = v[e] * rs * t[e];
      if (!kGateFirst) {
        Vec<T, V>::load(z + row * z_stride + c, t);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] *= (hn.sigmoid ? sigmoid_t<T>(t[e]) : silu_t<T>(t[e])) * hn.mult;
      }
      Vec<T, V>::store(out + row * (kGateFirst || !hn.out_stride ? width : hn.out_stride) + c, v);
    }
  }
}

// The second form of the above for runs of whole 16-byte pieces, up to 1,024 channels: L lanes (a power of two) per run,
// everything in registers.
template <typename T, int L, int kCh>
__global__ void __launch_bounds__(kNormThreads)
head_norm_gate_kernel(T* __restrict__ out, const T* __restrict__ y, int64_t y_stride, const T* __restrict__ z,
                      int64_t z_stride, const T* __restrict__ w, int64_t rows, int heads, int gs, float eps, const HeadNorm hn) {
  const int lane = threadIdx.x & (L - 1);
  const int64_t items = rows * heads, step = static_cast<int64_t>(gridDim.x) * (kNormThreads / L);
  for (int64_t i0 = static_cast<int64_t>(blockIdx.x) * (kNormThreads / L); i0 < items; i0 += step) {
    const int64_t i = i0 + threadIdx.x / L, row = i / heads;
    const int h = static_cast<int>(i - row * heads);
    const bool on = i < items;
    const float den = on && hn.den ? 1.f / hn.den[i] : 1.f;
    const T* wh = w + (hn.full_weight ? static_cast<int64_t>(h) * gs : 0);
    Raw8<T> a[kCh], b[kCh];
    float acc = 0.f;
#pragma unroll
    for (int k = 0; k < kCh; ++k) {
      const int c = (k * L + lane) * 8;
      if (on && c < gs) {
        a[k].load(y + row * y_stride + static_cast<int64_t>(h) * gs + c);
        b[k].load(z + row * z_stride + static_cast<int64_t>(h) * gs + c);
      }
    }
#pragma unroll
    for (int k = 0; k < kCh; ++k)
      if (on && (k * L + lane) * 8 < gs) {
        float v[8];
        a[k].get(v);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc = fmaf(v[e] * den, v[e] * den, acc);
      }
#pragma unroll
    for (int o = L / 2; o; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    const float rs = den / sqrtf(acc / static_cast<float>(gs) + eps);
#pragma unroll
    for (int k = 0; k < kCh; ++k) {
      const int c = (k * L + lane) * 8;
      if (on && c < gs) {
        float v[8], t[8], g[8];
        a[k].get(v);
        b[k].get(g);
        Vec<T, 8>::load(wh + c, t);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = v[e] * (rs * hn.mult) * t[e] * (hn.sigmoid ? sigmoid_t<T>(g[e]) : silu_t<T>(g[e]));
        Vec<T, 8>::store(out + row * (hn.out_stride ? hn.out_stride : static_cast<int64_t>(heads) * gs) + static_cast<int64_t>(h) * gs + c, v);
      }
    }
  }
}

// out = act(gate, y), see glu_act; row r of y is `heads` pieces of cols / heads elements, y_head_stride apart
template <typename T, int V>
__global__ void __launch_bounds__(kNormThreads)
gate_mul_kernel(T* __restrict__ out, const T* __restrict__ y, int64_t y_stride, int64_t y_head_stride, int head_cols,
                const T* __restrict__ gate, int64_t gate_stride, int act, float limit, int64_t rows, int cols) {
  const int per = cols / V;
  const int64_t total = rows * per;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * kNormThreads + threadIdx.x; i < total;
       i += static_cast<int64_t>(gridDim.x) * kNormThreads) {
    const int64_t row = i / per;
    const int c = static_cast<int>(i - row * per) * V, h = c / head_cols;
    float v[V], g[V];
    Vec<T, V>::load(y + row * y_stride + h * y_head_stride + (c - h * head_cols), v);
    Vec<T, V>::load(gate + row * gate_stride + c, g);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = glu_act<T>(act, g[e], v[e], limit);
    Vec<T, V>::store(out + row * cols + c, v);
  }
}

static size_t norm_smem(int width, int groups) {
  return sizeof(float) * (((width + 3) & ~3) + 2 * (groups < kNormWarps ? kNormWarps : groups));
}
template <typename K> static int allow_smem(K kernel, size_t bytes, const char* what) {
  if (bytes > 227 * 1024) return fail(MV_ERR_LIMIT, "%s: a row does not fit in shared memory", what);
  if (bytes > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes));
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
  }
  return MV_OK;
}

template <typename T, int V, int SRC>
static int launch_residual(const ResidualParams<T>& p, int64_t rows, cudaStream_t st) {
  const size_t smem = norm_smem(p.width, p.groups);
  const int rc = allow_smem(residual_norm_kernel<T, V, SRC>, smem, "residual_norm");
  if (rc) return rc;
  residual_norm_kernel<T, V, SRC><<<static_cast<unsigned>(rows), kNormThreads, smem, st>>>(p);
  return check_launch("residual_norm");
}
template <typename T, int SRC>
static int launch_residual_v(const ResidualParams<T>& p, int64_t rows, cudaStream_t st) {
  const int eb = sizeof(T);
  bool v8 = (p.width / p.groups) % 8 == 0 && aligned16(p.out) && aligned16(p.x) && aligned16(p.w_next) &&
            vec8_ok(p.y, p.y_stride, eb) && vec8_ok(p.gate, p.gate_stride, eb) && vec8_ok(p.gate_bias, 0, eb) &&
            vec8_ok(p.y2, p.y2_stride, eb) && vec8_ok(p.w_y, 0, eb) && vec8_ok(p.w_y2, 0, eb) && vec8_ok(p.w_post, 0, eb) && vec8_ok(p.embed, p.width, eb) && vec8_ok(p.shared, p.shared_stride, eb);
  if (v8 && p.groups <= kNormWarps) {
    const int lanes = kNormWarps / p.groups * 32, per = (p.width / p.groups / 8 + lanes - 1) / lanes;
    if (per <= 2) {
      if (per == 1) residual_norm_reg_kernel<T, SRC, 1><<<static_cast<unsigned>(rows), kNormThreads, 0, st>>>(p);
      else residual_norm_reg_kernel<T, SRC, 2><<<static_cast<unsigned>(rows), kNormThreads, 0, st>>>(p);
      return check_launch("residual_norm");
    }
  }
  return v8 ? launch_residual<T, 8, SRC>(p, rows, st) : launch_residual<T, 1, SRC>(p, rows, st);
}
static int check_norm(const char* what, int width, int groups, int dtype) {
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "%s: dtype %d", what, dtype);
  if (width <= 0 || groups <= 0 || width % groups) return fail(MV_ERR_SHAPE, "%s: width %d in %d groups", what, width, groups);
  return MV_OK;
}

}  // namespace mv

extern "C" int mv_embed_norm(void* out, float* x, const int64_t* ids, const void* embed, int64_t vocab,
                             const void* w_post, const void* w_next, int64_t rows, int width, int groups, float eps, int dtype,
                             void* stream) {
  using namespace mv;
  int rc = check_norm("embed_norm", width, groups, dtype);
  if (rc || rows == 0) return rc;
  if (!out || !x || !ids || !embed) return fail(MV_ERR_NULL, "embed_norm: null pointer");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    ResidualParams<T> p{};
    p.out = static_cast<T*>(out); p.x = x; p.ids = ids; p.embed = static_cast<const T*>(embed); p.vocab = vocab;
    p.w_post = static_cast<const T*>(w_post); p.w_next = static_cast<const T*>(w_next);
    p.width = width; p.groups = groups; p.eps = eps;
    return launch_residual_v<T, SRC_EMBED>(p, rows, static_cast<cudaStream_t>(stream));
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_gated_residual_norm(void* out, float* x, const void* y, int64_t y_stride, const void* gate,
                                      int64_t gate_stride, const void* gate_bias, const void* w_post,
                                      const void* w_next, float mult, int64_t rows, int width, int groups, float eps,
                                      int dtype, void* stream) {
  using namespace mv;
  int rc = check_norm("gated_residual_norm", width, groups, dtype);
  if (rc || rows == 0) return rc;
  if (!out || !x || !y || !w_post || (gate && !gate_bias))
    return fail(MV_ERR_NULL, "gated_residual_norm: null pointer");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    ResidualParams<T> p{};
    p.out = static_cast<T*>(out); p.x = x; p.y = static_cast<const T*>(y); p.y_stride = y_stride;
    p.gate = static_cast<const T*>(gate); p.gate_stride = gate_stride; p.gate_bias = static_cast<const T*>(gate_bias);
    p.w_post = static_cast<const T*>(w_post); p.w_next = static_cast<const T*>(w_next);
    p.mult = mult; p.width = width; p.groups = groups; p.eps = eps;
    return launch_residual_v<T, SRC_ROWS>(p, rows, static_cast<cudaStream_t>(stream));
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_pair_residual_norm(void* out, float* x, const void* a, int64_t a_stride, const void* w_a, const void* b,
                                     int64_t b_stride, const void* w_b, const void* w_post, const void* w_next,
                                     float mult, int64_t rows, int width, int groups, float eps, int dtype,
                                     void* stream) {
  using namespace mv;
  int rc = check_norm("pair_residual_norm", width, groups, dtype);
  if (rc || rows == 0) return rc;
  if (!out || !x || !a || !w_a || !b || !w_b || !w_post) return fail(MV_ERR_NULL, "pair_residual_norm: null pointer");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    ResidualParams<T> p{};
    p.out = static_cast<T*>(out); p.x = x; p.y = static_cast<const T*>(a); p.y_stride = a_stride;
    p.y2 = static_cast<const T*>(b); p.y2_stride = b_stride;
    p.w_y = static_cast<const T*>(w_a); p.w_y2 = static_cast<const T*>(w_b);
    p.w_post = static_cast<const T*>(w_post); p.w_next = static_cast<const T*>(w_next);
    p.mult = mult; p.width = width; p.groups = groups; p.eps = eps;
    return launch_residual_v<T, SRC_PAIR>(p, rows, static_cast<cudaStream_t>(stream));
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_moe_residual_norm(void* out, float* x, const void* expert_rows, const int32_t* pos,
                                    const float* top_weights, int top, const void* shared, int64_t shared_stride,
                                    const void* shared_gate, int64_t shared_gate_stride, const void* gate,
                                    int64_t gate_stride, const void* gate_bias, const void* w_post, const void* w_next,
                                    float mult, int64_t rows, int width, int groups, float eps, int dtype,
                                    void* stream) {
  using namespace mv;
  int rc = check_norm("moe_residual_norm", width, groups, dtype);
  if (rc || rows == 0) return rc;
  if (!out || !x || !expert_rows || !pos || !top_weights || !w_post || (gate && !gate_bias))
    return fail(MV_ERR_NULL, "moe_residual_norm: null pointer");
  if (top <= 0 || top > kMaxTop) return fail(MV_ERR_SHAPE, "moe_residual_norm: top %d", top);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    ResidualParams<T> p{};
    p.out = static_cast<T*>(out); p.x = x; p.y = static_cast<const T*>(expert_rows); p.y_stride = width;
    p.pos = pos; p.topw = top_weights; p.top = top;
    p.shared = static_cast<const T*>(shared); p.shared_stride = shared_stride;
    p.sg = static_cast<const T*>(shared_gate); p.sg_stride = shared_gate_stride;
    p.gate = static_cast<const T*>(gate); p.gate_stride = gate_stride; p.gate_bias = static_cast<const T*>(gate_bias);
    p.w_post = static_cast<const T*>(w_post); p.w_next = static_cast<const T*>(w_next);
    p.mult = mult; p.width = width; p.groups = groups; p.eps = eps;
    return launch_residual_v<T, SRC_EXPERTS>(p, rows, static_cast<cudaStream_t>(stream));
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

static int gated_norm(const char* what, bool gate_first, void* out, const void* y, int64_t y_stride, const void* z, int64_t z_stride,
                      const void* w, int64_t rows, int width, int groups, float eps, int dtype, void* stream, mv::HeadNorm hn = {nullptr, false, false, 1.f, 0}) {
  using namespace mv;
  int rc = check_norm(what, width, groups, dtype);
  if (rc || rows == 0) return rc;
  if (!out || !y || !z || !w) return fail(MV_ERR_NULL, "%s: null pointer", what);
  const size_t smem = norm_smem(width, groups);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int eb = sizeof(T);
    auto go = [&](auto kernel) {
      const int r = allow_smem(kernel, smem, what);
      if (r) return r;
      kernel<<<static_cast<unsigned>(rows), kNormThreads, smem, static_cast<cudaStream_t>(stream)>>>(
          static_cast<T*>(out), static_cast<const T*>(y), y_stride, static_cast<const T*>(z), z_stride,
          static_cast<const T*>(w), width, groups, eps, hn);
      return check_launch(what);
    };
    const bool v8 = (width / groups) % 8 == 0 && vec8_ok(out, hn.out_stride ? hn.out_stride : width, eb) && vec8_ok(y, y_stride, eb) && vec8_ok(z, z_stride, eb) &&
        aligned16(w);
    if (v8 && !gate_first && width / groups <= 1024) {
      const int gs = width / groups;
      auto lanes = [&](auto l, auto ch) {
        constexpr int L = decltype(l)::value;
        const int64_t blocks = (rows * groups + kNormThreads / L - 1) / (kNormThreads / L);
        head_norm_gate_kernel<T, L, decltype(ch)::value><<<static_cast<unsigned>(std::min<int64_t>(blocks, kNumSMs * 32)), kNormThreads, 0,
                                                           static_cast<cudaStream_t>(stream)>>>(
            static_cast<T*>(out), static_cast<const T*>(y), y_stride, static_cast<const T*>(z), z_stride, static_cast<const T*>(w),
            rows, groups, gs, eps, hn);
        return check_launch(what);
      };
      using std::integral_constant;
      if (gs <= 64) return lanes(integral_constant<int, 8>{}, integral_constant<int, 1>{});
      if (gs <= 128) return lanes(integral_constant<int, 16>{}, integral_constant<int, 1>{});
      if (gs <= 256) return lanes(integral_constant<int, 32>{}, integral_constant<int, 1>{});
      return lanes(integral_constant<int, 32>{}, integral_constant<int, 4>{});
    }
    if (v8)
      return gate_first ? go(gated_group_norm_kernel<T, 8, true>) : go(gated_group_norm_kernel<T, 8, false>);
    return gate_first ? go(gated_group_norm_kernel<T, 1, true>) : go(gated_group_norm_kernel<T, 1, false>);
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_gated_group_norm(void* out, const void* y, int64_t y_stride, const void* z, int64_t z_stride,
                                   const void* w, int64_t rows, int width, int groups, float eps, int dtype,
                                   void* stream) {
  return gated_norm("gated_group_norm", true, out, y, y_stride, z, z_stride, w, rows, width, groups, eps, dtype, stream);
}

extern "C" int mv_head_norm_gate(void* out, int64_t out_stride, const void* y, int64_t y_stride, const float* den, const void* z, int64_t z_stride,
                                 const void* w, int full_weight, int act, float mult, int64_t rows, int width, int heads,
                                 float eps, int dtype, void* stream) {
  if (act != MV_ACT_SILU && act != MV_ACT_SIGMOID) return mv::fail(MV_ERR_SHAPE, "head_norm_gate: activation %d", act);
  return gated_norm("head_norm_gate", false, out, y, y_stride, z, z_stride, w, rows, width, heads, eps, dtype, stream,
                    {den, full_weight != 0, act == MV_ACT_SIGMOID, mult, out_stride});
}

extern "C" int mv_gate_mul(void* out, const void* y, int64_t y_stride, int64_t y_head_stride, int heads,
                           const void* gate, int64_t gate_stride, int act, float limit, int64_t rows, int cols,
                           int dtype, void* stream) {
  using namespace mv;
  int rc = check_norm("gate_mul", cols, heads, dtype);
  if (rc || rows == 0) return rc;
  if (!out || !y || !gate) return fail(MV_ERR_NULL, "gate_mul: null pointer");
  if (act < 0 || act > MV_ACT_RELU) return fail(MV_ERR_SHAPE, "gate_mul: activation %d", act);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int eb = sizeof(T), hc = cols / heads;
    const bool v8 = hc % 8 == 0 && aligned16(out) && vec8_ok(y, y_stride, eb) && vec8_ok(y, y_head_stride, eb) &&
                    vec8_ok(gate, gate_stride, eb);
    const int64_t work = rows * (v8 ? cols / 8 : cols);
    const unsigned grid = static_cast<unsigned>(std::min<int64_t>((work + kNormThreads - 1) / kNormThreads, kNumSMs * 16));
    auto* o = static_cast<T*>(out);
    auto *a = static_cast<const T*>(y), *b = static_cast<const T*>(gate);
    auto st = static_cast<cudaStream_t>(stream);
    if (v8) gate_mul_kernel<T, 8><<<grid, kNormThreads, 0, st>>>(o, a, y_stride, y_head_stride, hc, b, gate_stride, act, limit, rows, cols);
    else gate_mul_kernel<T, 1><<<grid, kNormThreads, 0, st>>>(o, a, y_stride, y_head_stride, hc, b, gate_stride, act, limit, rows, cols);
    return check_launch("gate_mul");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}
