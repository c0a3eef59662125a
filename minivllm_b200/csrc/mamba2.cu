// State-space mixer (Mamba-2 / SSD) over a packed batch: short causal convolution, and the recurrence
//   S_t = exp(-exp(A_log) dt_t) S_{t-1} + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t
// per head, with the per-sequence state (the convolution's last inputs, and S in fp32) in slots that the engine
// assigns.  Sequence s of the batch has tokens cu[s] .. cu[s+1] and `start[s]` tokens behind it; start 0 means that
// the slot's contents belong to somebody else and count as zero.
//
// conv_silu_kernel      every token and channel of the step (reads the slot, does not change it); conv_silu_vec_kernel
//                       is the same with eight channels per thread and the taps in registers
// ssm_step_kernel       one token per sequence: convolution of the head's channels and one step of S, which is read
//                       and written once, in whole rows (HBM-bound: 8 * heads * N * P bytes per sequence)
// ssm_scan_kernel       token by token, S in shared memory: any sizes, bf16 or fp32
// conv_state_kernel     writes the slot's convolution inputs for the next step
#include <algorithm>
#include "vec.cuh"

namespace mv {

constexpr int kCvThreads = 128;
constexpr int kCvTokens = 8;    // tokens per CTA

// Input of the convolution `back` tokens before token j of the portion (0 before the start of the sequence).
template <typename T>
__device__ __forceinline__ float conv_input(const T* u, int64_t u_stride, int64_t first_row, int j, int c,
                                            const T* state, int hist, int channels) {
  if (j >= 0) return Elem<T>::to_f(u[(first_row + j) * u_stride + c]);
  return state && hist + j >= 0 ? Elem<T>::to_f(state[static_cast<int64_t>(hist + j) * channels + c]) : 0.f;
}

template <typename T>
__global__ void __launch_bounds__(kCvThreads)
conv_silu_kernel(T* __restrict__ out, const T* __restrict__ u, int64_t u_stride, const T* __restrict__ w,
                 const T* __restrict__ bias, int taps, int channels, const int32_t* __restrict__ cu, int num_seqs,
                 int64_t tokens, const int32_t* __restrict__ slots, const int32_t* __restrict__ start,
                 const T* __restrict__ state, int num_slots) {
  const int c = blockIdx.x * kCvThreads + threadIdx.x;
  if (c >= channels) return;
  const int hist = taps - 1;
  const float b = bias ? Elem<T>::to_f(bias[c]) : 0.f;
  const T* wc = w + static_cast<int64_t>(c) * taps;
  const int64_t t0 = static_cast<int64_t>(blockIdx.y) * kCvTokens;
  const int64_t t1 = min(t0 + kCvTokens, tokens);
  int s = -1, end = -1;
  int64_t first = 0;
  const T* st = nullptr;
  for (int64_t t = t0; t < t1; ++t) {
    if (t >= end) {
      s = seq_of_token(cu, num_seqs, static_cast<int>(t));
      first = cu ? cu[s] : t;
      end = cu ? cu[s + 1] : static_cast<int>(t) + 1;
      const int slot = slots[s];
      st = start[s] > 0 && slot >= 0 && slot < num_slots ? state + static_cast<int64_t>(slot) * hist * channels : nullptr;
    }
    const int j = static_cast<int>(t - first);
    float acc = b;
    for (int k = 0; k < taps; ++k)
      acc = fmaf(Elem<T>::to_f(wc[k]), conv_input(u, u_stride, first, j - hist + k, c, st, hist, channels), acc);
    out[t * channels + c] = Elem<T>::from_f(silu_t<T>(acc));
  }
}

// Eight channels per thread, up to kCvRun consecutive tokens, the last taps - 1 inputs kept in registers.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kCvThreads)
conv_silu_vec_kernel(T* __restrict__ out, const T* __restrict__ u, int64_t u_stride, const T* __restrict__ w,
                     const T* __restrict__ bias, int channels, const int32_t* __restrict__ cu, int num_seqs,
                     int64_t tokens, const int32_t* __restrict__ slots, const int32_t* __restrict__ start,
                     const T* __restrict__ state, int num_slots, int run) {
  constexpr int HIST = TAPS - 1;
  const int c = (blockIdx.x * kCvThreads + threadIdx.x) * 8;
  if (c >= channels) return;
  float wt[TAPS][8], b[8], win[HIST][8];
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    b[e] = bias ? Elem<T>::to_f(bias[c + e]) : 0.f;
#pragma unroll
    for (int k = 0; k < TAPS; ++k) wt[k][e] = Elem<T>::to_f(w[static_cast<int64_t>(c + e) * TAPS + k]);
  }
  const int64_t t0 = static_cast<int64_t>(blockIdx.y) * run, t1 = min(t0 + run, tokens);
  int64_t end = -1, ahead = -1;
  Raw8<T> raw[4];
  for (int64_t t = t0; t < t1; ++t) {
    if (t >= end) {                      // first token of this thread, or of a sequence: fetch what lies before it
      const int s = seq_of_token(cu, num_seqs, static_cast<int>(t));
      const int64_t first = cu ? cu[s] : t;
      end = cu ? cu[s + 1] : t + 1;
      const int slot = slots[s];
      const T* st = start[s] > 0 && slot >= 0 && slot < num_slots ? state + static_cast<int64_t>(slot) * HIST * channels : nullptr;
#pragma unroll
      for (int k = 0; k < HIST; ++k) {
        const int64_t j = t - first - HIST + k;
        if (j >= 0) {
          Vec<T, 8>::load(u + (first + j) * u_stride + c, win[k]);
        } else if (st && HIST + j >= 0) {
          Vec<T, 8>::load(st + (HIST + j) * channels + c, win[k]);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) win[k][e] = 0.f;
        }
      }
    }
    // four tokens at a time: their loads go out together, and the window needs no register moves
    if (t + 4 <= min(end, t1)) {
      float v[HIST + 4][8];
      if (ahead != t) {
#pragma unroll
        for (int k = 0; k < 4; ++k) raw[k].load(u + (t + k) * u_stride + c);
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) raw[k].get(v[HIST + k]);
      if (t + 8 <= min(end, t1)) {       // the next four are on their way while these are worked on
        ahead = t + 4;
#pragma unroll
        for (int k = 0; k < 4; ++k) raw[k].load(u + (t + 4 + k) * u_stride + c);
      }
#pragma unroll
      for (int k = 0; k < HIST; ++k)
#pragma unroll
        for (int e = 0; e < 8; ++e) v[k][e] = win[k][e];
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        float r[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          float a = b[e];
#pragma unroll
          for (int k = 0; k < TAPS; ++k) a = fmaf(wt[k][e], v[n + k][e], a);
          r[e] = silu_t<T>(a);
        }
        Vec<T, 8>::store(out + (t + n) * channels + c, r);
      }
#pragma unroll
      for (int k = 0; k < HIST; ++k)
#pragma unroll
        for (int e = 0; e < 8; ++e) win[k][e] = v[4 + k][e];
      t += 3;
      continue;
    }
    float v[8], r[8];
    Vec<T, 8>::load(u + t * u_stride + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      float a = b[e];
#pragma unroll
      for (int k = 0; k < HIST; ++k) a = fmaf(wt[k][e], win[k][e], a);
      r[e] = silu_t<T>(fmaf(wt[HIST][e], v[e], a));
#pragma unroll
      for (int k = 0; k + 1 < HIST; ++k) win[k][e] = win[k + 1][e];
      win[HIST - 1][e] = v[e];
    }
    Vec<T, 8>::store(out + t * channels + c, r);
  }
}

// One thread per (sequence, channel): shifts the slot's inputs.  Slots < 0 and sequences without tokens are left alone.
template <typename T>
__global__ void __launch_bounds__(kCvThreads)
conv_state_kernel(T* __restrict__ state, const T* __restrict__ u, int64_t u_stride, int taps, int channels,
                  const int32_t* __restrict__ cu, int num_seqs, const int32_t* __restrict__ slots,
                  const int32_t* __restrict__ start, int num_slots) {
  const int c = blockIdx.x * kCvThreads + threadIdx.x, s = blockIdx.y;
  if (c >= channels) return;
  const int slot = slots[s];
  const int st0 = start[s];
  if (slot < 0 || slot >= num_slots || st0 < 0) return;
  const int hist = taps - 1;
  const int64_t first = cu ? cu[s] : s;
  const int n = cu ? cu[s + 1] - cu[s] : 1;
  T* st = state + static_cast<int64_t>(slot) * hist * channels;
  for (int i = 0; i < hist; ++i) {          // ascending: entry i only needs entries above i
    const float v = conv_input(u, u_stride, first, n - hist + i, c, st0 > 0 ? st : nullptr, hist, channels);
    st[static_cast<int64_t>(i) * channels + c] = Elem<T>::from_f(v);
  }
}

constexpr int kScThreads = 256;

// One CTA per (sequence, head, block of value columns).  xbc: activated convolution output [x | B | C] per token.
template <typename T>
__global__ void __launch_bounds__(kScThreads)
ssm_scan_kernel(T* __restrict__ y, const T* __restrict__ xbc, const T* __restrict__ dt, int64_t dt_stride,
                const T* __restrict__ dt_bias, const T* __restrict__ A_log, const T* __restrict__ D,
                const int32_t* __restrict__ cu, int num_seqs, const int32_t* __restrict__ slots,
                const int32_t* __restrict__ start, float* __restrict__ state, int num_slots, int heads, int P, int N,
                int groups, int pb) {
  extern __shared__ __align__(16) float sm[];
  const int s = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * pb, pw = min(pb, P - p0);
  const int g = h / (heads / groups), inner = heads * P, channels = inner + 2 * groups * N;
  float* S = sm;                 // [N][pb]
  float* sB = S + N * pb;        // [N]
  float* sC = sB + N;            // [N]
  float* sx = sC + N;            // [pb]
  float* red = sx + pb;          // [splits][pb]
  const int splits = kScThreads / pb, p = threadIdx.x % pb, ns = threadIdx.x / pb;
  const bool on = ns < splits && p < pw;
  const int slot = slots[s], st0 = start[s];
  const bool live = slot >= 0 && slot < num_slots && st0 >= 0;
  const int64_t first = cu ? cu[s] : s;
  const int n_tok = cu ? cu[s + 1] - cu[s] : 1;
  float* gS = state + (static_cast<int64_t>(live ? slot : 0) * heads + h) * N * P;
  for (int i = threadIdx.x; i < N * pb; i += kScThreads) {
    const int n = i / pb, q = i - n * pb;
    S[i] = live && st0 > 0 && q < pw ? gS[static_cast<int64_t>(n) * P + p0 + q] : 0.f;
  }
  const float a = -expf(Elem<T>::to_f(A_log[h])), db = Elem<T>::to_f(dt_bias[h]), dd = Elem<T>::to_f(D[h]);
  for (int j = 0; j < n_tok; ++j) {
    const int64_t t = first + j;
    const T* row = xbc + t * channels;
    __syncthreads();
    for (int i = threadIdx.x; i < N; i += kScThreads) {
      sB[i] = Elem<T>::to_f(row[inner + g * N + i]);
      sC[i] = Elem<T>::to_f(row[inner + (groups + g) * N + i]);
    }
    for (int i = threadIdx.x; i < pw; i += kScThreads) sx[i] = Elem<T>::to_f(row[h * P + p0 + i]);
    __syncthreads();
    const float d = softplus_f(Elem<T>::to_f(dt[t * dt_stride + h]) + db), decay = expf(a * d);
    if (on) {
      const float dx = d * sx[p];
      float acc = 0.f;
      for (int n = ns; n < N; n += splits) {
        const float v = fmaf(decay, S[n * pb + p], sB[n] * dx);
        S[n * pb + p] = v;
        acc = fmaf(v, sC[n], acc);
      }
      red[ns * pb + p] = acc;
    }
    __syncthreads();
    if (on && ns == 0) {
      float acc = dd * sx[p];
      for (int k = 0; k < splits; ++k) acc += red[k * pb + p];
      y[t * inner + h * P + p0 + p] = Elem<T>::from_f(acc);
    }
  }
  __syncthreads();
  if (!live) return;
  for (int i = threadIdx.x; i < N * pb; i += kScThreads) {
    const int n = i / pb, q = i - n * pb;
    if (q < pw) gS[static_cast<int64_t>(n) * P + p0 + q] = S[i];
  }
}

constexpr int kStThreads = 256;
constexpr int kStBatch = 8;      // rows of S a thread has in flight

// One CTA per (sequence, head), one token: u is the row before the convolution.
template <typename T>
__global__ void __launch_bounds__(kStThreads)
ssm_step_kernel(T* __restrict__ y, const T* __restrict__ u, int64_t u_stride, const T* __restrict__ w,
                const T* __restrict__ bias, int taps, const T* __restrict__ conv_state, const T* __restrict__ dt,
                int64_t dt_stride, const T* __restrict__ dt_bias, const T* __restrict__ A_log, const T* __restrict__ D,
                const int32_t* __restrict__ slots, const int32_t* __restrict__ start, float* __restrict__ state,
                int num_slots, int heads, int P, int N, int groups) {
  extern __shared__ __align__(16) float sm[];
  const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int g = h / (heads / groups), inner = heads * P, channels = inner + 2 * groups * N, hist = taps - 1;
  float *sx = sm, *sB = sx + P, *sC = sB + N, *red = sC + N;      // red: [rows][P]
  const int slot = slots[s], st0 = start[s];
  const bool live = slot >= 0 && slot < num_slots && st0 >= 0;
  T* yr = y + static_cast<int64_t>(s) * inner + h * P;
  if (!live) {
    for (int i = tid; i < P; i += kStThreads) yr[i] = Elem<T>::from_f(0.f);
    return;
  }
  const int PQ = P / 4, rows = kStThreads / PQ, q = tid % PQ, r = tid / PQ;
  const bool on = r < rows;
  float4* gS = reinterpret_cast<float4*>(state + (static_cast<int64_t>(slot) * heads + h) * N * P);
  float4 v[kStBatch];
  auto fetch = [&](int n0) {
#pragma unroll
    for (int i = 0; i < kStBatch; ++i) {
      const int n = n0 + i * rows + r;
      v[i] = on && n < N && st0 > 0 ? gS[static_cast<int64_t>(n) * PQ + q] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  fetch(0);                                     // in flight while the convolution is computed
  const T* cs = conv_state + static_cast<int64_t>(slot) * hist * channels;
  for (int i = tid; i < P + 2 * N; i += kStThreads) {
    const int c = i < P ? h * P + i : i < P + N ? inner + g * N + i - P : inner + (groups + g) * N + i - P - N;
    float a = bias ? Elem<T>::to_f(bias[c]) : 0.f;
    const T* wc = w + static_cast<int64_t>(c) * taps;
    if (st0 > 0)
      for (int k = 0; k < hist; ++k) a = fmaf(Elem<T>::to_f(wc[k]), Elem<T>::to_f(cs[static_cast<int64_t>(k) * channels + c]), a);
    a = fmaf(Elem<T>::to_f(wc[hist]), Elem<T>::to_f(u[s * u_stride + c]), a);
    sm[i] = Elem<T>::to_f(Elem<T>::from_f(silu_t<T>(a)));       // rounded as the prompt path stores it
  }
  const float d = softplus_f(Elem<T>::to_f(dt[s * dt_stride + h]) + Elem<T>::to_f(dt_bias[h]));
  const float decay = expf(-expf(Elem<T>::to_f(A_log[h])) * d);
  __syncthreads();
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 x = on ? *reinterpret_cast<const float4*>(sx + q * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 dx = make_float4(d * x.x, d * x.y, d * x.z, d * x.w);
  for (int n0 = 0; n0 < N; n0 += kStBatch * rows) {
    if (n0) fetch(n0);
#pragma unroll
    for (int i = 0; i < kStBatch; ++i) {
      const int n = n0 + i * rows + r;
      if (on && n < N) {
        const float b = sB[n], c = sC[n];
        v[i].x = fmaf(decay, v[i].x, b * dx.x);
        v[i].y = fmaf(decay, v[i].y, b * dx.y);
        v[i].z = fmaf(decay, v[i].z, b * dx.z);
        v[i].w = fmaf(decay, v[i].w, b * dx.w);
        gS[static_cast<int64_t>(n) * PQ + q] = v[i];
        acc.x = fmaf(v[i].x, c, acc.x);
        acc.y = fmaf(v[i].y, c, acc.y);
        acc.z = fmaf(v[i].z, c, acc.z);
        acc.w = fmaf(v[i].w, c, acc.w);
      }
    }
  }
  if (on) {
    float* o = red + r * P + q * 4;
    o[0] = acc.x; o[1] = acc.y; o[2] = acc.z; o[3] = acc.w;
  }
  __syncthreads();
  for (int i = tid; i < P; i += kStThreads) {
    float a = Elem<T>::to_f(D[h]) * sx[i];
    for (int k = 0; k < rows; ++k) a += red[k * P + i];
    yr[i] = Elem<T>::from_f(a);
  }
}

}  // namespace mv

static int check_ssm(const char* what, int dtype, int num_seqs, int channels, int taps) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "%s: dtype %d", what, dtype);
  if (num_seqs < 0 || channels <= 0 || taps <= 0) return fail(MV_ERR_SHAPE, "%s: %d sequences, %d channels, %d taps", what, num_seqs, channels, taps);
  return MV_OK;
}

extern "C" int mv_conv_silu(void* out, const void* u, int64_t u_stride, const void* w, const void* bias, int taps,
                            int channels, const int32_t* cu, int num_seqs, int64_t tokens, const int32_t* slots,
                            const int32_t* start, const void* state, int num_slots, int dtype, void* stream) {
  using namespace mv;
  const int rc = check_ssm("conv_silu", dtype, num_seqs, channels, taps);
  if (rc || tokens == 0 || num_seqs == 0) return rc;
  if (!out || !u || !w || !slots || !start || (taps > 1 && !state)) return fail(MV_ERR_NULL, "conv_silu: null pointer");
  const dim3 grid((channels + kCvThreads - 1) / kCvThreads, static_cast<unsigned>((tokens + kCvTokens - 1) / kCvTokens));
  if (grid.y > 65535) return fail(MV_ERR_LIMIT, "conv_silu: %lld tokens", static_cast<long long>(tokens));
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int eb = sizeof(T);
    if (taps >= 2 && taps <= 4 && channels % 8 == 0 && vec8_ok(out, channels, eb) && vec8_ok(u, u_stride, eb) && vec8_ok(state, channels, eb)) {
      const int len = tokens > 4096 ? 32 : tokens > 512 ? 8 : 2;      // longer runs re-read fewer inputs
      const dim3 vg((channels / 8 + kCvThreads - 1) / kCvThreads, static_cast<unsigned>((tokens + len - 1) / len));
      auto go = [&](auto kernel) {
        kernel<<<vg, kCvThreads, 0, static_cast<cudaStream_t>(stream)>>>(
            static_cast<T*>(out), static_cast<const T*>(u), u_stride, static_cast<const T*>(w), static_cast<const T*>(bias),
            channels, cu, num_seqs, tokens, slots, start, static_cast<const T*>(state), num_slots, len);
        return check_launch("conv_silu");
      };
      return taps == 2 ? go(conv_silu_vec_kernel<T, 2>) : taps == 3 ? go(conv_silu_vec_kernel<T, 3>) : go(conv_silu_vec_kernel<T, 4>);
    }
    conv_silu_kernel<T><<<grid, kCvThreads, 0, static_cast<cudaStream_t>(stream)>>>(
        static_cast<T*>(out), static_cast<const T*>(u), u_stride, static_cast<const T*>(w), static_cast<const T*>(bias),
        taps, channels, cu, num_seqs, tokens, slots, start, static_cast<const T*>(state), num_slots);
    return check_launch("conv_silu");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_conv_state_update(void* state, const void* u, int64_t u_stride, int taps, int channels,
                                    const int32_t* cu, int num_seqs, const int32_t* slots, const int32_t* start,
                                    int num_slots, int dtype, void* stream) {
  using namespace mv;
  const int rc = check_ssm("conv_state_update", dtype, num_seqs, channels, taps);
  if (rc || num_seqs == 0 || taps == 1) return rc;
  if (!state || !u || !slots || !start) return fail(MV_ERR_NULL, "conv_state_update: null pointer");
  const dim3 grid((channels + kCvThreads - 1) / kCvThreads, num_seqs);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    conv_state_kernel<T><<<grid, kCvThreads, 0, static_cast<cudaStream_t>(stream)>>>(
        static_cast<T*>(state), static_cast<const T*>(u), u_stride, taps, channels, cu, num_seqs, slots, start, num_slots);
    return check_launch("conv_state_update");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_ssm_scan(void* y, const void* xbc, const void* dt, int64_t dt_stride, const void* dt_bias,
                           const void* A_log, const void* D, const int32_t* cu, int num_seqs, const int32_t* slots,
                           const int32_t* start, float* state, int num_slots, int heads, int vdim, int state_dim,
                           int groups, int dtype, void* stream) {
  using namespace mv;
  const int rc = check_ssm("ssm_scan", dtype, num_seqs, heads, 1);
  if (rc || num_seqs == 0) return rc;
  if (vdim <= 0 || state_dim <= 0 || groups <= 0 || heads % groups)
    return fail(MV_ERR_SHAPE, "ssm_scan: heads %d groups %d vdim %d state %d", heads, groups, vdim, state_dim);
  if (!y || !xbc || !dt || !dt_bias || !A_log || !D || !slots || !start || !state)
    return fail(MV_ERR_NULL, "ssm_scan: null pointer");
  int pb = std::min(vdim, 64);
  while (pb > 1 && static_cast<int64_t>(state_dim) * pb > 48000) pb /= 2;
  const int splits = kScThreads / pb;
  const size_t smem = sizeof(float) * (static_cast<size_t>(state_dim) * pb + 2 * state_dim + pb + splits * pb);
  if (smem > 227 * 1024) return fail(MV_ERR_LIMIT, "ssm_scan: state %d too large", state_dim);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const cudaError_t e = cudaFuncSetAttribute(ssm_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "ssm_scan: %s", cudaGetErrorString(e));
    const dim3 grid(num_seqs, heads, (vdim + pb - 1) / pb);
    ssm_scan_kernel<T><<<grid, kScThreads, smem, static_cast<cudaStream_t>(stream)>>>(
        static_cast<T*>(y), static_cast<const T*>(xbc), static_cast<const T*>(dt), dt_stride,
        static_cast<const T*>(dt_bias), static_cast<const T*>(A_log), static_cast<const T*>(D), cu, num_seqs, slots,
        start, state, num_slots, heads, vdim, state_dim, groups, pb);
    return check_launch("ssm_scan");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_ssm_step(void* y, const void* u, int64_t u_stride, const void* w, const void* bias, int taps,
                           const void* conv_state, const void* dt, int64_t dt_stride, const void* dt_bias,
                           const void* A_log, const void* D, int num_seqs, const int32_t* slots, const int32_t* start,
                           float* state, int num_slots, int heads, int vdim, int state_dim, int groups, int dtype,
                           void* stream) {
  using namespace mv;
  const int rc = check_ssm("ssm_step", dtype, num_seqs, heads, taps);
  if (rc || num_seqs == 0) return rc;
  if (vdim <= 0 || vdim % 4 || vdim > 4 * kStThreads || state_dim <= 0 || state_dim % 4 || groups <= 0 || heads % groups)
    return fail(MV_ERR_SHAPE, "ssm_step: heads %d groups %d vdim %d state %d", heads, groups, vdim, state_dim);
  if (!y || !u || !w || (taps > 1 && !conv_state) || !dt || !dt_bias || !A_log || !D || !slots || !start || !state)
    return fail(MV_ERR_NULL, "ssm_step: null pointer");
  if (!aligned16(state)) return fail(MV_ERR_ALIGN, "ssm_step: state");
  const int rows = kStThreads / (vdim / 4);
  const size_t smem = sizeof(float) * (static_cast<size_t>(vdim) + 2 * state_dim + rows * vdim);
  if (smem > 48 * 1024) return fail(MV_ERR_LIMIT, "ssm_step: state %d", state_dim);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    ssm_step_kernel<T><<<dim3(num_seqs, heads), kStThreads, smem, static_cast<cudaStream_t>(stream)>>>(
        static_cast<T*>(y), static_cast<const T*>(u), u_stride, static_cast<const T*>(w), static_cast<const T*>(bias), taps,
        static_cast<const T*>(conv_state), static_cast<const T*>(dt), dt_stride, static_cast<const T*>(dt_bias),
        static_cast<const T*>(A_log), static_cast<const T*>(D), slots, start, state, num_slots, heads, vdim, state_dim, groups);
    return check_launch("ssm_step");
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}
