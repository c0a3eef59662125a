// The gated delta rule over a packed batch, the state in slots: see state_scan.cuh.
#include "state_scan.cuh"

extern "C" int mv_delta_scan(void* out, int64_t out_stride, const void* qkv, int64_t stride, const void* beta,
                             const void* a, int64_t ba_stride, const void* A_log, const void* dt_bias, const int32_t* cu,
                             int num_seqs, const int32_t* slots, const int32_t* start, float* state, int num_slots,
                             int heads, int kv_heads, int dim, int vdim, float q_scale, const void* conv_w, int taps,
                             const void* conv_state, const void* gate, int64_t gate_stride, const void* norm_w, float eps,
                             int dtype, void* stream) {
  using namespace mv;
  const int rc = check_scan("delta_scan", dtype, num_seqs, heads, kv_heads, dim, vdim);
  if (rc || num_seqs == 0) return rc;
  if (!out || !qkv || !beta || !a || !A_log || !dt_bias || !slots || !start || !state) return fail(MV_ERR_NULL, "delta_scan: null pointer");
  if (!cu && (!gate || !norm_w || !conv_w || taps <= 0 || (taps > 1 && !conv_state))) return fail(MV_ERR_NULL, "delta_scan: null pointer");
  if (!aligned16(state)) return fail(MV_ERR_ALIGN, "delta_scan: state");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto c = [](const void* x) { return static_cast<const T*>(x); };
    ScanParams<T> p{};
    p.out = static_cast<T*>(out); p.out_stride = out_stride;
    p.q = c(qkv); p.k = p.q + kv_heads * dim; p.v = p.k + kv_heads * dim; p.stride = stride;
    p.beta = c(beta); p.a = c(a); p.gate_stride = ba_stride; p.A_log = c(A_log); p.dt_bias = c(dt_bias);
    p.cu = cu; p.slots = slots; p.start = start; p.state = state; p.num_slots = num_slots;
    p.heads = heads; p.kv_heads = kv_heads; p.K = dim; p.V = vdim; p.q_scale = q_scale;
    p.gate = c(gate); p.out_gate_stride = gate_stride; p.norm_w = c(norm_w); p.eps = eps;
    p.conv_w = c(conv_w); p.conv_state = c(conv_state); p.taps = taps; p.channels = 2 * kv_heads * dim + heads * vdim;
    auto st = static_cast<cudaStream_t>(stream);
    return cu ? run_scan<SK_DELTA, T>(p, num_seqs, st) : run_step<SK_DELTA, T>(p, num_seqs, st);
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}
