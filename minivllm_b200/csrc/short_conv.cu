// Short causal depthwise convolution over a packed batch, followed by silu or added to its own input, with the last inputs of
// every sequence in slots that the engine assigns.  Sequence s of the batch has tokens cu[s] .. cu[s+1] and `start[s]` tokens behind it;
// start 0 means that the slot's contents belong to somebody else and count as zero.
//
// conv_kernel           every token and channel of the step (reads the slot, does not change it); conv_vec_kernel
//                       is the same with eight channels per thread and the taps in registers
// conv_state_kernel     writes the slot's inputs for the next step
#include <algorithm>
#include "vec.cuh"

namespace mv {

constexpr int kCvThreads = 128;
constexpr int kCvTokens = 8;    // tokens per CTA
enum { CV_SILU = 0, CV_ADD = 1 };

// What becomes of a convolution's result; v: the newest input.
template <typename T, int OP> __device__ __forceinline__ float conv_result(float acc, float v) {
  return OP == CV_SILU ? silu_t<T>(acc) : acc + v;
}

// Input of the convolution `back` tokens before token j of the portion (0 before the start of the sequence).
template <typename T>
__device__ __forceinline__ float conv_input(const T* u, int64_t u_stride, int64_t first_row, int j, int c,
                                            const T* state, int hist, int channels) {
  if (j >= 0) return Elem<T>::to_f(u[(first_row + j) * u_stride + c]);
  return state && hist + j >= 0 ? Elem<T>::to_f(state[static_cast<int64_t>(hist + j) * channels + c]) : 0.f;
}

template <typename T, int OP>
__global__ void __launch_bounds__(kCvThreads)
conv_kernel(T* __restrict__ out, const T* __restrict__ u, int64_t u_stride, const T* __restrict__ w,
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
    out[t * channels + c] = Elem<T>::from_f(conv_result<T, OP>(acc, conv_input(u, u_stride, first, j, c, st, hist, channels)));
  }
}

// Eight channels per thread, up to kCvRun consecutive tokens, the last taps - 1 inputs kept in registers.
template <typename T, int TAPS, int OP>
__global__ void __launch_bounds__(kCvThreads)
conv_vec_kernel(T* __restrict__ out, const T* __restrict__ u, int64_t u_stride, const T* __restrict__ w,
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
          r[e] = conv_result<T, OP>(a, v[n + HIST][e]);
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
      r[e] = conv_result<T, OP>(fmaf(wt[HIST][e], v[e], a), v[e]);
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

}  // namespace mv

static int check_conv(const char* what, int dtype, int num_seqs, int channels, int taps) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "%s: dtype %d", what, dtype);
  if (num_seqs < 0 || channels <= 0 || taps <= 0) return fail(MV_ERR_SHAPE, "%s: %d sequences, %d channels, %d taps", what, num_seqs, channels, taps);
  return MV_OK;
}

template <int OP>
static int run_conv(const char* what, void* out, const void* u, int64_t u_stride, const void* w, const void* bias, int taps,
                    int channels, const int32_t* cu, int num_seqs, int64_t tokens, const int32_t* slots,
                    const int32_t* start, const void* state, int num_slots, int dtype, void* stream) {
  using namespace mv;
  const int rc = check_conv(what, dtype, num_seqs, channels, taps);
  if (rc || tokens == 0 || num_seqs == 0) return rc;
  if (!out || !u || !w || !slots || !start || (taps > 1 && !state)) return fail(MV_ERR_NULL, "%s: null pointer", what);
  const dim3 grid((channels + kCvThreads - 1) / kCvThreads, static_cast<unsigned>((tokens + kCvTokens - 1) / kCvTokens));
  if (grid.y > 65535) return fail(MV_ERR_LIMIT, "%s: %lld tokens", what, static_cast<long long>(tokens));
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
        return check_launch(what);
      };
      return taps == 2 ? go(conv_vec_kernel<T, 2, OP>) : taps == 3 ? go(conv_vec_kernel<T, 3, OP>) : go(conv_vec_kernel<T, 4, OP>);
    }
    conv_kernel<T, OP><<<grid, kCvThreads, 0, static_cast<cudaStream_t>(stream)>>>(
        static_cast<T*>(out), static_cast<const T*>(u), u_stride, static_cast<const T*>(w), static_cast<const T*>(bias),
        taps, channels, cu, num_seqs, tokens, slots, start, static_cast<const T*>(state), num_slots);
    return check_launch(what);
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_conv_silu(void* out, const void* u, int64_t u_stride, const void* w, const void* bias, int taps,
                            int channels, const int32_t* cu, int num_seqs, int64_t tokens, const int32_t* slots,
                            const int32_t* start, const void* state, int num_slots, int dtype, void* stream) {
  return run_conv<mv::CV_SILU>("conv_silu", out, u, u_stride, w, bias, taps, channels, cu, num_seqs, tokens, slots, start, state, num_slots, dtype, stream);
}

extern "C" int mv_conv_add(void* out, const void* u, int64_t u_stride, const void* w, const void* bias, int taps,
                           int channels, const int32_t* cu, int num_seqs, int64_t tokens, const int32_t* slots,
                           const int32_t* start, const void* state, int num_slots, int dtype, void* stream) {
  return run_conv<mv::CV_ADD>("conv_add", out, u, u_stride, w, bias, taps, channels, cu, num_seqs, tokens, slots, start, state, num_slots, dtype, stream);
}

extern "C" int mv_conv_state_update(void* state, const void* u, int64_t u_stride, int taps, int channels,
                                    const int32_t* cu, int num_seqs, const int32_t* slots, const int32_t* start,
                                    int num_slots, int dtype, void* stream) {
  using namespace mv;
  const int rc = check_conv("conv_state_update", dtype, num_seqs, channels, taps);
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
