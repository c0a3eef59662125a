// Gated linear attention over a packed batch, the state in slots: see state_scan.cuh.
#include "state_scan.cuh"

extern "C" int mv_gla_scan(void* out, int64_t out_stride, const void* q, const void* k, const void* v, int64_t stride,
                           const void* z, int64_t z_stride, float tau, const int32_t* cu, int num_seqs,
                           const int32_t* slots, const int32_t* start, float* state, int num_slots, int heads, int dim,
                           int vdim, float q_scale, const void* gate, int64_t gate_stride, const void* norm_w, float eps,
                           int dtype, void* stream) {
  using namespace mv;
  const int rc = check_scan("gla_scan", dtype, num_seqs, heads, heads, dim, vdim);
  if (rc || num_seqs == 0) return rc;
  if (!(tau > 0.f)) return fail(MV_ERR_SHAPE, "gla_scan: tau %f", tau);
  if (!out || !q || !k || !v || !z || !slots || !start || !state || (!cu && (!gate || !norm_w))) return fail(MV_ERR_NULL, "gla_scan: null pointer");
  if (!aligned16(state)) return fail(MV_ERR_ALIGN, "gla_scan: state");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto c = [](const void* x) { return static_cast<const T*>(x); };
    ScanParams<T> p{};
    p.out = static_cast<T*>(out); p.out_stride = out_stride;
    p.q = c(q); p.k = c(k); p.v = c(v); p.stride = stride; p.z = c(z); p.z_stride = z_stride; p.inv_tau = 1.f / tau;
    p.cu = cu; p.slots = slots; p.start = start; p.state = state; p.num_slots = num_slots;
    p.heads = heads; p.kv_heads = heads; p.K = dim; p.V = vdim; p.q_scale = q_scale;
    p.gate = c(gate); p.out_gate_stride = gate_stride; p.norm_w = c(norm_w); p.eps = eps;
    auto st = static_cast<cudaStream_t>(stream);
    return cu ? run_scan<SK_GLA, T>(p, num_seqs, st) : run_step<SK_GLA, T>(p, num_seqs, st);
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}
