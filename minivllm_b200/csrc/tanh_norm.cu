// What stands between two sublayers of a decoder with an fp32 residual stream and an element-wise norm (Dynamic Tanh,
// h = tanh(alpha x) w + b): one launch adds a sublayer's result (or takes the embedding row and its position's sinusoids, or
// sums the pieces of a mixture of experts), and writes the next sublayer's input.  In front of a mixer that looks one token
// back it also writes the mixtures h + (h' - h) mu of a token's input with the one before it (h'; zeros before the first),
// kept per sequence in slots.  Plus element-wise activations of ungated feed-forwards.
//
// HBM-bound.  A thread walks along the rows of its channels.  With mixtures the stream goes to another buffer: a thread that
// starts in the middle of a sequence forms the input before its first one again, from the stream as it was.
#include <algorithm>
#include "vec.cuh"

namespace mv {

constexpr int kTnThreads = 128;
enum { TN_EMBED = 0, TN_ROWS = 1, TN_EXPERTS = 2 };

template <typename T> struct TanhStepParams {
  T* out;                                      // (rows, width)
  const float* x_in; float* x_out;             // (rows, width)
  const int64_t* ids; const T* embed; int64_t vocab; const int64_t* positions; const double* inv_freq;   // TN_EMBED; inv_freq null: no sinusoids
  const T* y; int64_t y_stride;                // TN_ROWS: sublayer result; TN_EXPERTS: expert rows (sorted)
  const int32_t* pos; const float* topw; int top;
  float alpha; const T *w, *b;
  const T* mu; T* mixed; int mixes;            // (mixes, width), (mixes, rows, width)
  T* kept; const int32_t *slots, *start; int num_slots;      // (num_slots, width)
  const int32_t* cu; int num_seqs;             // null: one token each
  int64_t rows; int width;
};

// tanh; where the result is rounded to 16 bits, from the special-function unit (absolute error of fp32, relative far below the rounding).
template <typename T> __device__ __forceinline__ float tanh_t(float z) {
  if (sizeof(T) != 2) return tanhf(z);
  const float far = 1.f - __fdividef(2.f, __expf(2.f * z) + 1.f), near = z * fmaf(z * z, -0.33333333f, 1.f);
  return fabsf(z) < 0.02f ? near : far;
}

template <typename T, int V, int SRC, bool kMix>
__global__ void __launch_bounds__(kTnThreads) tanh_step_kernel(const TanhStepParams<T> p, int run) {
  const int c = (blockIdx.x * kTnThreads + threadIdx.x) * V;
  if (c >= p.width) return;
  float w[V], b[V];
  Vec<T, V>::load(p.w + c, w);
  Vec<T, V>::load(p.b + c, b);
  auto stream = [&](int64_t row, float (&v)[V]) {        // the stream behind the sublayer
    if (SRC == TN_EMBED) {
      int64_t token = p.ids[row];
      if (token < 0 || token >= p.vocab) token = 0;      // placeholder rows of a padded batch
      Vec<T, V>::load(p.embed + token * p.width + c, v);
      if (p.inv_freq) {
        const double at = static_cast<double>(p.positions[row]);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          double a = at * p.inv_freq[(c + e) / 2];
          a -= rint(a * 0.15915494309189535) * 6.283185307179586;
          v[e] += (c + e) & 1 ? cosf(static_cast<float>(a)) : sinf(static_cast<float>(a));
        }
      }
    } else {
      Vec<float, V>::load(p.x_in + row * p.width + c, v);
      float t[V];
      if (SRC == TN_ROWS) {
        Vec<T, V>::load(p.y + row * p.y_stride + c, t);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) t[e] = 0.f;
        constexpr int kAtOnce = 4;
        for (int k0 = 0; k0 < p.top; k0 += kAtOnce) {
          float u[kAtOnce][V];
#pragma unroll
          for (int k = 0; k < kAtOnce; ++k)
            if (k0 + k < p.top) Vec<T, V>::load(p.y + static_cast<int64_t>(p.pos[row * p.top + k0 + k]) * p.y_stride + c, u[k]);
#pragma unroll
          for (int k = 0; k < kAtOnce; ++k)
            if (k0 + k < p.top) {
              const float f = p.topw[row * p.top + k0 + k];
#pragma unroll
              for (int e = 0; e < V; ++e) t[e] = fmaf(f, u[k][e], t[e]);
            }
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += t[e];
    }
  };
  auto norm = [&](const float (&v)[V], float (&h)[V]) {  // as the next sublayer reads it
#pragma unroll
    for (int e = 0; e < V; ++e) h[e] = Elem<T>::to_f(Elem<T>::from_f(fmaf(tanh_t<T>(p.alpha * v[e]), w[e], b[e])));
  };
  const int64_t r0 = static_cast<int64_t>(blockIdx.y) * run, r1 = min(r0 + run, p.rows);
  int64_t end = -1;
  float before[V];
  T* kept = nullptr;
  for (int64_t row = r0; row < r1; ++row) {
    float v[V], h[V];
    if (kMix && row >= end) {            // first token of this thread, or of a sequence
      const int s = seq_of_token(p.cu, p.num_seqs, static_cast<int>(row));
      const int64_t first = p.cu ? p.cu[s] : row;
      end = p.cu ? p.cu[s + 1] : row + 1;
      const int slot = p.slots[s], st0 = p.start[s];
      const bool live = slot >= 0 && slot < p.num_slots && st0 >= 0;
      kept = live ? p.kept + static_cast<int64_t>(slot) * p.width + c : nullptr;
      if (row > first) {
        stream(row - 1, v);
        norm(v, before);
      } else if (live && st0 > 0) {
        Vec<T, V>::load(kept, before);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) before[e] = 0.f;
      }
      if (end - first > 1) kept = nullptr;     // longer portions: the slot moves on after this launch
    }
    stream(row, v);
    norm(v, h);
    Vec<float, V>::store(p.x_out + row * p.width + c, v);
    Vec<T, V>::store(p.out + row * p.width + c, h);
    if (kMix) {
      if (kept) Vec<T, V>::store(kept, h);
      for (int m = 0; m < p.mixes; ++m) {
        float mu[V], x[V];
        Vec<T, V>::load(p.mu + static_cast<int64_t>(m) * p.width + c, mu);
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = fmaf(before[e] - h[e], mu[e], h[e]);
        Vec<T, V>::store(p.mixed + (m * p.rows + row) * p.width + c, x);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) before[e] = h[e];
    }
  }
}

// z > 0: a z^2 + z / 2;  z <= 0: b (e^z - 1 - z) + z / 2.  Near zero e^z - 1 - z from its series.
__device__ __forceinline__ float xielu_f(float z, float a, float b) {
  float s = 2.48015873e-5f;
  s = fmaf(s, z, 1.98412698e-4f);
  s = fmaf(s, z, 1.38888889e-3f);
  s = fmaf(s, z, 8.33333333e-3f);
  s = fmaf(s, z, 4.16666667e-2f);
  s = fmaf(s, z, 1.66666667e-1f);
  s = fmaf(s, z, 0.5f);
  const float far = expf(z) - 1.f - z, low = z > -0.5f ? s * z * z : far;
  return fmaf(0.5f, z, z > 0.f ? a * z * z : b * low);
}

enum { EW_XIELU = 0, EW_TANH = 1 };
template <typename TI, typename T, int V, int OP>
__global__ void __launch_bounds__(256) elementwise_kernel(T* __restrict__ out, const TI* __restrict__ y, int64_t y_stride, float a, float b, int64_t rows, int cols) {
  const int per = cols / V;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < rows * per; i += static_cast<int64_t>(gridDim.x) * 256) {
    const int64_t row = i / per;
    const int c = static_cast<int>(i - row * per) * V;
    float v[V];
    Vec<TI, V>::load(y + row * y_stride + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = OP == EW_XIELU ? xielu_f(v[e], a, b) : tanhf(v[e]);
    Vec<T, V>::store(out + row * cols + c, v);
  }
}

template <int OP, typename TI, typename T>
static int launch_elementwise(const char* what, void* out, const void* y, int64_t y_stride, float a, float b, int64_t rows, int cols, cudaStream_t st) {
  auto* o = static_cast<T*>(out);
  auto* in = static_cast<const TI*>(y);
  const bool v8 = cols % 8 == 0 && aligned16(out) && vec8_ok(y, y_stride, sizeof(TI));
  const int64_t work = rows * (v8 ? cols / 8 : cols);
  const unsigned grid = static_cast<unsigned>(std::min<int64_t>((work + 255) / 256, kNumSMs * 16));
  if (v8) elementwise_kernel<TI, T, 8, OP><<<grid, 256, 0, st>>>(o, in, y_stride, a, b, rows, cols);
  else elementwise_kernel<TI, T, 1, OP><<<grid, 256, 0, st>>>(o, in, y_stride, a, b, rows, cols);
  return check_launch(what);
}

template <typename T, int SRC> static int launch_tanh_step(const TanhStepParams<T>& p, cudaStream_t st) {
  const int eb = sizeof(T);
  const bool v8 = p.width % 8 == 0 && aligned16(p.out) && aligned16(p.x_in) && aligned16(p.x_out) && aligned16(p.w) && aligned16(p.b) &&
                  vec8_ok(p.y, p.y_stride, eb) && aligned16(p.embed) && aligned16(p.mu) && aligned16(p.mixed) && aligned16(p.kept);
  // longer runs read the norm's weights (and, with mixtures, a row) less often; short ones fill the GPU
  const int64_t cols = (p.width / (v8 ? 8 : 1) + kTnThreads - 1) / kTnThreads;
  const int run = static_cast<int>(std::max<int64_t>(1, std::min<int64_t>(16, p.rows * cols / (kNumSMs * 16))));
  const int64_t gy = (p.rows + run - 1) / run;
  if (gy > 65535) return fail(MV_ERR_LIMIT, "tanh_step: %lld rows", static_cast<long long>(p.rows));
  const dim3 grid(static_cast<unsigned>(cols), static_cast<unsigned>(gy));
  auto go = [&](auto kernel) {
    kernel<<<grid, kTnThreads, 0, st>>>(p, run);
    return check_launch("tanh_step");
  };
  if (p.mixes) return v8 ? go(tanh_step_kernel<T, 8, SRC, true>) : go(tanh_step_kernel<T, 1, SRC, true>);
  return v8 ? go(tanh_step_kernel<T, 8, SRC, false>) : go(tanh_step_kernel<T, 1, SRC, false>);
}

}  // namespace mv

extern "C" int mv_tanh_step(void* out, float* x_out, const float* x_in, const int64_t* ids, const void* embed, int64_t vocab,
                            const int64_t* positions, const double* inv_freq, const void* y, int64_t y_stride,
                            const int32_t* pos, const float* top_weights, int top, float alpha, const void* w, const void* b,
                            void* mixed, const void* mu, int mixes, void* kept, const int32_t* slots, const int32_t* start,
                            int num_slots, const int32_t* cu, int num_seqs, int64_t rows, int width, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "tanh_step: dtype %d", dtype);
  if (rows < 0 || width <= 0 || mixes < 0 || (pos && top <= 0)) return fail(MV_ERR_SHAPE, "tanh_step: width %d, %d mixtures, top %d", width, mixes, top);
  if (rows == 0) return MV_OK;
  if (!out || !x_out || !w || !b || (ids ? !embed || (inv_freq && !positions) : !x_in || !y) || (pos && !top_weights) ||
      (mixes && (!mixed || !mu || !kept || !slots || !start)))
    return fail(MV_ERR_NULL, "tanh_step: null pointer");
  if (mixes && !ids && x_in == x_out) return fail(MV_ERR_SHAPE, "tanh_step: mixtures want the new stream in another buffer");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto k = [](const void* x) { return static_cast<const T*>(x); };
    TanhStepParams<T> p{};
    p.out = static_cast<T*>(out); p.x_in = x_in; p.x_out = x_out; p.ids = ids; p.embed = k(embed); p.vocab = vocab; p.positions = positions;
    p.inv_freq = inv_freq; p.y = k(y); p.y_stride = y_stride; p.pos = pos; p.topw = top_weights; p.top = top; p.alpha = alpha; p.w = k(w);
    p.b = k(b); p.mu = k(mu); p.mixed = static_cast<T*>(mixed); p.mixes = mixes; p.kept = static_cast<T*>(kept); p.slots = slots;
    p.start = start; p.num_slots = num_slots; p.cu = cu; p.num_seqs = num_seqs; p.rows = rows; p.width = width;
    auto st = static_cast<cudaStream_t>(stream);
    if (ids) return launch_tanh_step<T, TN_EMBED>(p, st);
    return pos ? launch_tanh_step<T, TN_EXPERTS>(p, st) : launch_tanh_step<T, TN_ROWS>(p, st);
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}

extern "C" int mv_xielu(void* out, const void* y, int64_t y_stride, float a, float b, int64_t rows, int cols, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "xielu: dtype %d", dtype);
  if (rows < 0 || cols <= 0) return fail(MV_ERR_SHAPE, "xielu: %d columns", cols);
  if (rows == 0) return MV_OK;
  if (!out || !y) return fail(MV_ERR_NULL, "xielu: null pointer");
  auto st = static_cast<cudaStream_t>(stream);
  return dtype == MV_F32 ? launch_elementwise<EW_XIELU, float, float>("xielu", out, y, y_stride, a, b, rows, cols, st)
                         : launch_elementwise<EW_XIELU, __nv_bfloat16, __nv_bfloat16>("xielu", out, y, y_stride, a, b, rows, cols, st);
}

extern "C" int mv_tanh_rows(void* out, const float* y, int64_t y_stride, int64_t rows, int cols, int dtype, void* stream) {
  using namespace mv;
  if (dtype != MV_BF16 && dtype != MV_F32) return fail(MV_ERR_DTYPE, "tanh_rows: dtype %d", dtype);
  if (rows < 0 || cols <= 0) return fail(MV_ERR_SHAPE, "tanh_rows: %d columns", cols);
  if (rows == 0) return MV_OK;
  if (!out || !y) return fail(MV_ERR_NULL, "tanh_rows: null pointer");
  auto st = static_cast<cudaStream_t>(stream);
  return dtype == MV_F32 ? launch_elementwise<EW_TANH, float, float>("tanh_rows", out, y, y_stride, 0.f, 0.f, rows, cols, st)
                         : launch_elementwise<EW_TANH, float, __nv_bfloat16>("tanh_rows", out, y, y_stride, 0.f, 0.f, rows, cols, st);
}
