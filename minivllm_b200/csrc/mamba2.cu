// State-space mixer (Mamba-2 / SSD) over a packed batch: the recurrence
//   S_t = exp(-exp(A_log) dt_t) S_{t-1} + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t
// per head, with the per-sequence state (S in fp32; the convolution's last inputs, short_conv.cu) in slots that the engine
// assigns.  Sequence s of the batch has tokens cu[s] .. cu[s+1] and `start[s]` tokens behind it; start 0 means that
// the slot's contents belong to somebody else and count as zero.
//
// ssm_step_kernel       one token per sequence: convolution of the head's channels and one step of S, which is read
//                       and written once, in whole rows (HBM-bound: 8 * heads * N * P bytes per sequence)
// ssm_scan_kernel       token by token, S in shared memory: any sizes, bf16 or fp32
#include <algorithm>
#include "vec.cuh"

namespace mv {

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
