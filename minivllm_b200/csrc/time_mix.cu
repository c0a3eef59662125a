// Time mixing (a decay per channel from the token, a bonus for the token's own entry) over a packed batch, the state in slots:
// see state_scan.cuh.
#include "state_scan.cuh"

extern "C" int mv_time_scan(void* out, int64_t out_stride, const void* r, const void* k, const void* v, int64_t stride,
                            const float* z, int64_t z_stride, const void* w0, const void* bonus, const int32_t* cu,
                            int num_seqs, const int32_t* slots, const int32_t* start, float* state, int num_slots, int heads,
                            int dim, int vdim, const void* gate, int64_t gate_stride, const void* norm_w, float eps,
                            float out_scale, int dtype, void* stream) {
  using namespace mv;
  const int rc = check_scan("time_scan", dtype, num_seqs, heads, heads, dim, vdim);
  if (rc || num_seqs == 0) return rc;
  if (!out || !r || !k || !v || !z || !w0 || !bonus || !slots || !start || !state || (!cu && (!gate || !norm_w)))
    return fail(MV_ERR_NULL, "time_scan: null pointer");
  if (!aligned16(state)) return fail(MV_ERR_ALIGN, "time_scan: state");
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto c = [](const void* x) { return static_cast<const T*>(x); };
    ScanParams<T> p{};
    p.out = static_cast<T*>(out); p.out_stride = out_stride;
    p.q = c(r); p.k = c(k); p.v = c(v); p.stride = stride; p.zf = z; p.zf_stride = z_stride; p.w0 = c(w0); p.bonus = c(bonus);
    p.cu = cu; p.slots = slots; p.start = start; p.state = state; p.num_slots = num_slots;
    p.heads = heads; p.kv_heads = heads; p.K = dim; p.V = vdim; p.q_scale = 1.f;
    p.gate = c(gate); p.out_gate_stride = gate_stride; p.norm_w = c(norm_w); p.eps = eps; p.out_scale = out_scale;
    auto st = static_cast<cudaStream_t>(stream);
    return cu ? run_scan<SK_TIME, T>(p, num_seqs, st) : run_step<SK_TIME, T>(p, num_seqs, st);
  };
  return dtype == MV_F32 ? run(float{}) : run(__nv_bfloat16{});
}
