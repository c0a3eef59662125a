// Residual streams: a decoder keeps several fp32 copies x_1 .. x_s of the residual instead of one.  One launch stands between
// two sublayers:
//   x_t <- sum_s mix[s][t] x_s + out[t] y        (all new streams from the old ones, y the result of the sublayer before)
//   u = sum_s in[s] x_s                          (in null: the plain sum, in front of the head)
//   h = norm(u)                                  (layer norm with weight and bias; without a bias an RMS norm)
// or, with token ids, sets every stream to the embedding row first.
//
// A causal convolution over time may follow the norm: h_t + sum_j taps[j] h_(t - n + 1 + j).  Rows that are one-token sequences
// (the first conv_rows) get it here, from the inputs kept in their slot, which move on in the same launch; the other rows leave
// h in `raw` for mv_conv_add, which needs their neighbours.
//
// HBM-bound: a row moves 8 * streams * width + 4 * width bytes (bf16).  A CTA owns a row.
#include <algorithm>
#include <type_traits>
#include "vec.cuh"

namespace mv {

constexpr int kSmThreads = 256, kSmWarps = kSmThreads / 32;
constexpr int kMaxStreams = 16;
constexpr int kSmHist = 3;             // kept inputs that the register form fetches ahead

template <typename T> struct StreamParams {
  T *out, *raw;                        // (rows, width): rows below conv_rows go to out, the others to raw (from its first row)
  float* x;                            // (rows, streams, width)
  const int64_t* ids; const T* embed; int64_t vocab;
  const T* y; int64_t y_stride;
  const T *mix, *w_out, *w_in;         // (streams, streams) [from][to], (streams), (streams)
  const T *norm_w, *norm_b;
  int64_t conv_rows;
  const T* taps_t; int taps;           // (taps, width)
  T* conv_state;                       // (num_slots, taps - 1, width)
  const int32_t *slots, *start; int num_slots;
  int width, streams;
  float eps;
};

// Sum over the block, the same for every thread; `part` is used once per call.
__device__ __forceinline__ float block_sum(float v, float* part) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int w = 0; w < kSmWarps; ++w) s += part[w];
  return s;
}

template <typename T> __device__ __forceinline__ int64_t embed_row(const StreamParams<T>& p, int64_t row) {
  const int64_t t = p.ids[row];
  return t < 0 || t >= p.vocab ? 0 : t;          // placeholder rows of a padded batch
}

// Width a multiple of eight: the row in registers, kCh pieces of eight channels per thread.
template <typename T, int S, int kCh>
__global__ void __launch_bounds__(kSmThreads) stream_step_kernel(const StreamParams<T> p) {
  __shared__ float part[2][kSmWarps];
  const int64_t row = blockIdx.x;
  const int W = p.width;
  const bool conv = p.taps > 0 && row < p.conv_rows;
  int slot = -1, st0 = 0;
  if (conv) {
    slot = p.slots[row];
    st0 = p.start[row];
    if (slot >= p.num_slots || st0 < 0) slot = -1;
  }
  T* kept = p.conv_state + (slot >= 0 ? static_cast<int64_t>(slot) * (p.taps - 1) * W : 0);
  const bool ahead = conv && p.taps - 1 <= kSmHist;
  float mix[S][S], wo[S], wi[S], in_sum = 0.f;
#pragma unroll
  for (int s = 0; s < S; ++s) {
    wi[s] = p.w_in ? Elem<T>::to_f(p.w_in[s]) : 1.f;
    in_sum += wi[s];
    if (!p.ids) {
      wo[s] = Elem<T>::to_f(p.w_out[s]);
#pragma unroll
      for (int t = 0; t < S; ++t) mix[s][t] = Elem<T>::to_f(p.mix[s * S + t]);
    }
  }
  float* x = p.x + row * S * W;
  const int64_t token = p.ids ? embed_row(p, row) : 0;
  float u[kCh][8], sum = 0.f;
  Raw8<T> hist[kCh][kSmHist];
#pragma unroll
  for (int k = 0; k < kCh; ++k) {
    const int c = (k * kSmThreads + threadIdx.x) * 8;
    if (c >= W) continue;
    if (ahead) {
#pragma unroll
      for (int j = 0; j < kSmHist; ++j)
        if (j < p.taps - 1 && slot >= 0 && st0 > 0) hist[k][j].load(kept + static_cast<int64_t>(j) * W + c);
    }
    if (p.ids) {
      float e[8];
      Vec<T, 8>::load(p.embed + token * W + c, e);
#pragma unroll
      for (int s = 0; s < S; ++s) Vec<float, 8>::store(x + s * W + c, e);
#pragma unroll
      for (int i = 0; i < 8; ++i) u[k][i] = in_sum * e[i];
    } else {
      float old[S][8], y[8];
#pragma unroll
      for (int s = 0; s < S; ++s) Vec<float, 8>::load(x + s * W + c, old[s]);
      Vec<T, 8>::load(p.y + row * p.y_stride + c, y);
#pragma unroll
      for (int i = 0; i < 8; ++i) u[k][i] = 0.f;
#pragma unroll
      for (int t = 0; t < S; ++t) {
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          v[i] = wo[t] * y[i];
#pragma unroll
          for (int s = 0; s < S; ++s) v[i] = fmaf(mix[s][t], old[s][i], v[i]);
          u[k][i] = fmaf(wi[t], v[i], u[k][i]);
        }
        Vec<float, 8>::store(x + t * W + c, v);
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) sum += u[k][i];
  }
  const float mean = p.norm_b ? block_sum(sum, part[0]) / static_cast<float>(W) : 0.f;
  sum = 0.f;
#pragma unroll
  for (int k = 0; k < kCh; ++k)
    if ((k * kSmThreads + static_cast<int>(threadIdx.x)) * 8 < W) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        u[k][i] -= mean;
        sum = fmaf(u[k][i], u[k][i], sum);
      }
    }
  const float rs = 1.f / sqrtf(block_sum(sum, part[1]) / static_cast<float>(W) + p.eps);
  T* dst = row < p.conv_rows ? p.out + row * W : p.raw + (row - p.conv_rows) * W;
#pragma unroll
  for (int k = 0; k < kCh; ++k) {
    const int c = (k * kSmThreads + threadIdx.x) * 8;
    if (c >= W) continue;
    float w[8], b[8] = {};
    Vec<T, 8>::load(p.norm_w + c, w);
    if (p.norm_b) Vec<T, 8>::load(p.norm_b + c, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) w[i] = fmaf(u[k][i] * rs, w[i], b[i]);
    if (conv) {
      // the convolution sees h as it is kept, rounded
      float acc[8], t[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) w[i] = Elem<T>::to_f(Elem<T>::from_f(w[i]));
      Vec<T, 8>::load(p.taps_t + static_cast<int64_t>(p.taps - 1) * W + c, t);
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i] = fmaf(t[i], w[i], w[i]);
      if (slot >= 0) {
        if (ahead) {
#pragma unroll
          for (int j = 0; j < kSmHist; ++j)
            if (j < p.taps - 1) {
              float v[8] = {};
              if (st0 > 0) hist[k][j].get(v);
              Vec<T, 8>::load(p.taps_t + static_cast<int64_t>(j) * W + c, t);
#pragma unroll
              for (int i = 0; i < 8; ++i) acc[i] = fmaf(t[i], v[i], acc[i]);
              if (j > 0) Vec<T, 8>::store(kept + static_cast<int64_t>(j - 1) * W + c, v);
            }
        } else {
          for (int j = 0; j < p.taps - 1; ++j) {
            float v[8] = {};
            if (st0 > 0) Vec<T, 8>::load(kept + static_cast<int64_t>(j) * W + c, v);
            Vec<T, 8>::load(p.taps_t + static_cast<int64_t>(j) * W + c, t);
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[i] = fmaf(t[i], v[i], acc[i]);
            if (j > 0) Vec<T, 8>::store(kept + static_cast<int64_t>(j - 1) * W + c, v);
          }
        }
        if (p.taps > 1) Vec<T, 8>::store(kept + static_cast<int64_t>(p.taps - 2) * W + c, w);
      }
      Vec<T, 8>::store(dst + c, acc);
    } else {
      Vec<T, 8>::store(dst + c, w);
    }
  }
}

// Any sizes: u in shared memory, one channel per thread at a time.
template <typename T>
__global__ void __launch_bounds__(kSmThreads) stream_step_any_kernel(const StreamParams<T> p) {
  extern __shared__ __align__(16) float s_u[];
  __shared__ float part[2][kSmWarps];
  __shared__ float mix[kMaxStreams * kMaxStreams], wo[kMaxStreams], wi[kMaxStreams];
  const int64_t row = blockIdx.x;
  const int W = p.width, S = p.streams, tid = threadIdx.x;
  if (tid < S) {
    wi[tid] = p.w_in ? Elem<T>::to_f(p.w_in[tid]) : 1.f;
    wo[tid] = p.ids ? 0.f : Elem<T>::to_f(p.w_out[tid]);
  }
  if (!p.ids)
    for (int i = tid; i < S * S; i += kSmThreads) mix[i] = Elem<T>::to_f(p.mix[i]);
  __syncthreads();
  float* x = p.x + row * S * W;
  const int64_t token = p.ids ? embed_row(p, row) : 0;
  float sum = 0.f;
  for (int c = tid; c < W; c += kSmThreads) {
    float u = 0.f;
    if (p.ids) {
      const float e = Elem<T>::to_f(p.embed[token * W + c]);
      for (int s = 0; s < S; ++s) {
        x[s * W + c] = e;
        u = fmaf(wi[s], e, u);
      }
    } else {
      const float y = Elem<T>::to_f(p.y[row * p.y_stride + c]);
      float old[kMaxStreams];
      for (int s = 0; s < S; ++s) old[s] = x[s * W + c];
      for (int t = 0; t < S; ++t) {
        float v = wo[t] * y;
        for (int s = 0; s < S; ++s) v = fmaf(mix[s * S + t], old[s], v);
        x[t * W + c] = v;
        u = fmaf(wi[t], v, u);
      }
    }
    s_u[c] = u;
    sum += u;
  }
  const float mean = p.norm_b ? block_sum(sum, part[0]) / static_cast<float>(W) : 0.f;
  sum = 0.f;
  for (int c = tid; c < W; c += kSmThreads) {
    const float d = s_u[c] - mean;
    sum = fmaf(d, d, sum);
  }
  const float rs = 1.f / sqrtf(block_sum(sum, part[1]) / static_cast<float>(W) + p.eps);
  const bool conv = p.taps > 0 && row < p.conv_rows;
  int slot = -1, st0 = 0;
  if (conv) {
    slot = p.slots[row];
    st0 = p.start[row];
    if (slot >= p.num_slots || st0 < 0) slot = -1;
  }
  T* dst = row < p.conv_rows ? p.out + row * W : p.raw + (row - p.conv_rows) * W;
  for (int c = tid; c < W; c += kSmThreads) {
    const float h = fmaf((s_u[c] - mean) * rs, Elem<T>::to_f(p.norm_w[c]), p.norm_b ? Elem<T>::to_f(p.norm_b[c]) : 0.f);
    const T ht = Elem<T>::from_f(h);
    if (!conv) {
      dst[c] = ht;
      continue;
    }
    const float hr = Elem<T>::to_f(ht);
    float acc = fmaf(Elem<T>::to_f(p.taps_t[static_cast<int64_t>(p.taps - 1) * W + c]), hr, hr);
    if (slot >= 0) {
      T* kept = p.conv_state + static_cast<int64_t>(slot) * (p.taps - 1) * W + c;
      for (int j = 0; j < p.taps - 1; ++j) {
        const T v = st0 > 0 ? kept[static_cast<int64_t>(j) * W] : Elem<T>::from_f(0.f);
        acc = fmaf(Elem<T>::to_f(p.taps_t[static_cast<int64_t>(j) * W + c]), Elem<T>::to_f(v), acc);
        if (j > 0) kept[static_cast<int64_t>(j - 1) * W] = v;
      }
      if (p.taps > 1) kept[static_cast<int64_t>(p.taps - 2) * W] = ht;
    }
    dst[c] = Elem<T>::from_f(acc);
  }
}

template <typename T, int S> static bool launch_streams_reg(const StreamParams<T>& p, int64_t rows, cudaStream_t st) {
  const int per = (p.width / 8 + kSmThreads - 1) / kSmThreads;
  const unsigned g = static_cast<unsigned>(rows);
  if (per == 1) stream_step_kernel<T, S, 1><<<g, kSmThreads, 0, st>>>(p);
  else if (per == 2) stream_step_kernel<T, S, 2><<<g, kSmThreads, 0, st>>>(p);
  else if (per <= 4) stream_step_kernel<T, S, 4><<<g, kSmThreads, 0, st>>>(p);
  else return false;
  return true;
}

template <typename T> static int launch_streams(const StreamParams<T>& p, int64_t rows, cudaStream_t st) {
  const int eb = sizeof(T);
  const bool v8 = p.width % 8 == 0 && aligned16(p.out) && aligned16(p.raw) && aligned16(p.x) && aligned16(p.embed) &&
                  vec8_ok(p.y, p.y_stride, eb) && aligned16(p.norm_w) && aligned16(p.norm_b) && aligned16(p.taps_t) && aligned16(p.conv_state);
  bool done = false;
  if (v8) {
    if (p.streams == 1) done = launch_streams_reg<T, 1>(p, rows, st);
    else if (p.streams == 2) done = launch_streams_reg<T, 2>(p, rows, st);
    else if (p.streams == 3) done = launch_streams_reg<T, 3>(p, rows, st);
    else if (p.streams == 4) done = launch_streams_reg<T, 4>(p, rows, st);
  }
  if (!done) {
    const size_t smem = sizeof(float) * p.width;
    if (smem > 200 * 1024) return fail(MV_ERR_LIMIT, "stream_step: width %d", p.width);
    const cudaError_t e = cudaFuncSetAttribute(stream_step_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return fail(MV_ERR_CUDA, "stream_step: %s", cudaGetErrorString(e));
    stream_step_any_kernel<T><<<static_cast<unsigned>(rows), kSmThreads, smem, st>>>(p);
  }
  return check_launch("stream_step");
}

}  // namespace mv

extern "C" int mv_stream_step(void* out, void* raw, float* x, const int64_t* ids, const void* embed, int64_t vocab,
                              const void* y, int64_t y_stride, const void* mix, const void* w_out, const void* w_in,
                              const void* norm_w, const void* norm_b, const void* taps_t, int taps, void* conv_state,
                              const int32_t* slots, const int32_t* start, int num_slots, int64_t conv_rows, int64_t rows,
                              int width, int streams, float eps, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "stream_step: dtype %d", dtype);
  if (rows < 0 || conv_rows < 0 || conv_rows > rows || width <= 0 || streams <= 0 || taps < 0)
    return fail(MV_ERR_SHAPE, "stream_step: %lld rows, width %d, %d streams, %d taps", static_cast<long long>(rows), width, streams, taps);
  if (streams > kMaxStreams) return fail(MV_ERR_LIMIT, "stream_step: %d streams (at most %d)", streams, kMaxStreams);
  if (rows == 0) return MV_OK;
  if (!x || !norm_w || (conv_rows > 0 && !out) || (conv_rows < rows && !raw)) return fail(MV_ERR_NULL, "stream_step: null pointer");
  if (ids ? !embed || vocab <= 0 : !y || !mix || !w_out) return fail(MV_ERR_NULL, "stream_step: null source");
  if (taps > 0 && conv_rows > 0 && (!taps_t || !slots || !start || (taps > 1 && !conv_state))) return fail(MV_ERR_NULL, "stream_step: null convolution");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto c = [](const void* q) { return static_cast<const T*>(q); };
    StreamParams<T> p{};
    p.out = static_cast<T*>(out); p.raw = static_cast<T*>(raw); p.x = x; p.ids = ids; p.embed = c(embed); p.vocab = vocab;
    p.y = c(y); p.y_stride = y_stride; p.mix = c(mix); p.w_out = c(w_out); p.w_in = c(w_in); p.norm_w = c(norm_w); p.norm_b = c(norm_b);
    p.conv_rows = conv_rows; p.taps_t = c(taps_t); p.taps = taps; p.conv_state = static_cast<T*>(conv_state);
    p.slots = slots; p.start = start; p.num_slots = num_slots; p.width = width; p.streams = streams; p.eps = eps;
    return launch_streams(p, rows, static_cast<cudaStream_t>(stream));
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}
