// Matrix memory with exponential gates (mLSTM) over a packed batch, the state in slots: the chain of running maxima here, the
// recurrence token by token in state_scan.cuh.
#include "state_scan.cuh"

namespace mv {

// One CTA per (sequence, head): m' = max(f + m, i) token by token.  A run of tokens acts on m as m -> max(m + F, A), F the sum
// of the f's, and runs compose: a thread takes kMgRun tokens, a scan over the CTA gives it the m in front of them.
constexpr int kMgRun = 4, kMgThreads = 512, kMgWarps = kMgThreads / 32, kMgTile = kMgRun * kMgThreads;

template <typename T> __global__ void __launch_bounds__(kMgThreads) mlstm_gates_kernel(const ScanParams<T> p, float4* __restrict__ chain) {
  __shared__ float2 s_run[kMgWarps];     // (F, A) of a warp's tokens
  __shared__ float s_last[kMgWarps];     // m behind them
  const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int first = p.cu[s], n_tok = p.cu[s + 1] - first;
  if (n_tok <= 0) return;
  const int slot = p.slots[s], st0 = p.start[s];
  const bool live = slot >= 0 && slot < p.num_slots && st0 >= 0;
  float* gm = p.m_state + static_cast<int64_t>(live ? slot : 0) * p.heads + h;
  float m = live && st0 > 0 ? *gm : 0.f;
  const float ib = Elem<T>::to_f(p.i_b[h]), fb = Elem<T>::to_f(p.f_b[h]);
  float zi[kMgRun], zf[kMgRun];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int e = 0; e < kMgRun; ++e) {
      const int t = t0 + tid * kMgRun + e;
      const float* z = p.gates + static_cast<int64_t>(first + (t < n_tok ? t : 0)) * p.gates_stride + h;
      zi[e] = z[0];
      zf[e] = z[p.heads];
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < n_tok; t0 += kMgTile) {
    const int mine = t0 + tid * kMgRun;
    float i[kMgRun], f[kMgRun], F = 0.f, A = -INFINITY;
#pragma unroll
    for (int e = 0; e < kMgRun; ++e) {
      i[e] = -INFINITY;                  // past the end: m stays
      f[e] = 0.f;
    }
    if (mine - lane * kMgRun < n_tok) {  // the warp has tokens
#pragma unroll
      for (int e = 0; e < kMgRun; ++e) {
        if (mine + e < n_tok) {
          i[e] = mem_log_input(zi[e] + ib, p.cap);
          f[e] = mem_log_forget(zf[e] + fb, p.cap);
        }
        A = fmaxf(A + f[e], i[e]);
        F += f[e];
      }
      if (t0 + kMgTile < n_tok) fetch(t0 + kMgTile);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float Fb = __shfl_up_sync(0xffffffffu, F, o), Ab = __shfl_up_sync(0xffffffffu, A, o);
        if (lane >= o) {
          A = fmaxf(Ab + F, A);
          F += Fb;
        }
      }
    }
    if (lane == 31) s_run[warp] = make_float2(F, A);
    __syncthreads();
    float at = m;
    for (int w = 0; w < warp; ++w) at = fmaxf(at + s_run[w].x, s_run[w].y);
    const float Fb = __shfl_up_sync(0xffffffffu, F, 1), Ab = __shfl_up_sync(0xffffffffu, A, 1);
    if (lane > 0) at = fmaxf(at + Fb, Ab);
    float after[kMgRun];
#pragma unroll
    for (int e = 0; e < kMgRun; ++e) after[e] = at = fmaxf(f[e] + at, i[e]);
    if (lane == 31) s_last[warp] = at;
    __syncthreads();
    // what a token continues is what the token before it left, to the last bit
    float before = __shfl_up_sync(0xffffffffu, at, 1);
    if (lane == 0) before = warp == 0 ? m : s_last[warp - 1];
#pragma unroll
    for (int e = 0; e < kMgRun; ++e) {
      if (mine + e < n_tok) chain[static_cast<int64_t>(first + mine + e) * p.heads + h] = make_float4(i[e], f[e], before, after[e]);
      if (mine + e == n_tok - 1 && live) *gm = after[e];
      before = after[e];
    }
    m = s_last[kMgWarps - 1];
    __syncthreads();                     // the tables are free again
  }
}

template <typename F> static int by_dtype(int dtype, F&& f) { return dtype == MV_F32 ? f(float{}) : f(__nv_bfloat16{}); }

}  // namespace mv

extern "C" int mv_mlstm_gates(float* chain, const float* gates, int64_t gates_stride, const void* i_b, const void* f_b,
                              float cap, const int32_t* cu, int num_seqs, const int32_t* slots, const int32_t* start,
                              float* m_state, int num_slots, int heads, int dtype, void* stream) {
  using namespace mv;
  const int rc = check_scan("mlstm_gates", dtype, num_seqs, heads, heads, 1, 1);
  if (rc || num_seqs == 0) return rc;
  if (!(cap > 0.f)) return fail(MV_ERR_SHAPE, "mlstm_gates: cap %f", cap);
  if (!chain || !gates || !i_b || !f_b || !cu || !slots || !start || !m_state) return fail(MV_ERR_NULL, "mlstm_gates: null pointer");
  if (!aligned16(chain)) return fail(MV_ERR_ALIGN, "mlstm_gates: chain");
  return by_dtype(dtype, [&](auto tag) {
    using T = decltype(tag);
    ScanParams<T> p{};
    p.gates = gates; p.gates_stride = gates_stride; p.i_b = static_cast<const T*>(i_b); p.f_b = static_cast<const T*>(f_b); p.cap = cap;
    p.cu = cu; p.slots = slots; p.start = start; p.m_state = m_state; p.num_slots = num_slots; p.heads = heads;
    mlstm_gates_kernel<T><<<dim3(num_seqs, heads), kMgThreads, 0, static_cast<cudaStream_t>(stream)>>>(p, reinterpret_cast<float4*>(chain));
    return check_launch("mlstm_gates");
  });
}

extern "C" int mv_mlstm_scan(void* out, int64_t out_stride, float* den, const void* q, const void* k, const void* v,
                             int64_t stride, const float* chain, const int32_t* cu, int num_seqs, const int32_t* slots,
                             const int32_t* start, float* S, float* n, int num_slots, int heads, int dim, int vdim,
                             float q_scale, int dtype, void* stream) {
  using namespace mv;
  const int rc = check_scan("mlstm_scan", dtype, num_seqs, heads, heads, dim, vdim);
  if (rc || num_seqs == 0) return rc;
  if (!out || !den || !q || !k || !v || !chain || !cu || !slots || !start || !S || !n) return fail(MV_ERR_NULL, "mlstm_scan: null pointer");
  if (!aligned16(S) || !aligned16(chain)) return fail(MV_ERR_ALIGN, "mlstm_scan: state");
  return by_dtype(dtype, [&](auto tag) {
    using T = decltype(tag);
    auto c = [](const void* x) { return static_cast<const T*>(x); };
    ScanParams<T> p{};
    p.out = static_cast<T*>(out); p.out_stride = out_stride; p.q = c(q); p.k = c(k); p.v = c(v); p.stride = stride;
    p.chain = reinterpret_cast<const float4*>(chain); p.den = den; p.n_state = n;
    p.cu = cu; p.slots = slots; p.start = start; p.state = S; p.num_slots = num_slots;
    p.heads = heads; p.kv_heads = heads; p.K = dim; p.V = vdim; p.q_scale = q_scale;
    return run_scan<SK_MLSTM, T>(p, num_seqs, static_cast<cudaStream_t>(stream));
  });
}

extern "C" int mv_mlstm_step(void* out, int64_t out_stride, const void* q, const void* k, const void* v, int64_t stride,
                             const void* x, int64_t x_stride, const void* gates_w, int width, const void* i_b, const void* f_b,
                             float cap, int num_seqs, const int32_t* slots, const int32_t* start, float* S, float* n, float* m,
                             int num_slots, int heads, int dim, int vdim, float q_scale, const void* gate,
                             int64_t gate_stride, const void* norm_w, float eps, int dtype, void* stream) {
  using namespace mv;
  const int rc = check_scan("mlstm_step", dtype, num_seqs, heads, heads, dim, vdim);
  if (rc || num_seqs == 0) return rc;
  if (!(cap > 0.f) || width <= 0) return fail(MV_ERR_SHAPE, "mlstm_step: cap %f, width %d", cap, width);
  if (!out || !q || !k || !v || !x || !gates_w || !i_b || !f_b || !slots || !start || !S || !n || !m || !gate || !norm_w)
    return fail(MV_ERR_NULL, "mlstm_step: null pointer");
  if (!aligned16(S)) return fail(MV_ERR_ALIGN, "mlstm_step: state");
  return by_dtype(dtype, [&](auto tag) {
    using T = decltype(tag);
    auto c = [](const void* t) { return static_cast<const T*>(t); };
    ScanParams<T> p{};
    p.out = static_cast<T*>(out); p.out_stride = out_stride; p.q = c(q); p.k = c(k); p.v = c(v); p.stride = stride;
    p.x = c(x); p.x_stride = x_stride; p.gates_w = c(gates_w); p.width = width; p.i_b = c(i_b); p.f_b = c(f_b); p.cap = cap; p.n_state = n; p.m_state = m;
    p.slots = slots; p.start = start; p.state = S; p.num_slots = num_slots;
    p.heads = heads; p.kv_heads = heads; p.K = dim; p.V = vdim; p.q_scale = q_scale;
    p.gate = c(gate); p.out_gate_stride = gate_stride; p.norm_w = c(norm_w); p.eps = eps;
    return run_step<SK_MLSTM, T>(p, num_seqs, static_cast<cudaStream_t>(stream));
  });
}
