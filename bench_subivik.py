"""`bench.py --workload subivik`: throughput of the Subivik family beside the Fozerax family (the closest one: attention beside a
recurrence on a matrix state in one layer, mixtures of experts) at equal size, and every kernel of the family against its
roofline, beside the like kernel of Fozerax.

Sizes: random weights, four layers (talking-heads attention beside time mixing, and differential attention, in turn, the second
of the latter on the first one's keys and values), mixtures of experts without a shared one; the Fozerax model of a size has the
same width, layer count, vocabulary, heads and experts.  Prefill is one wave of 16 prompts x 1,024 tokens, decode the captured
graph with 64 sequences behind 1,024-token contexts; both timed on the device with CUDA events around the engine's own step,
per-step inputs of more than the L2 size (weights, cache and state).
"""
import torch

import bench_fozerax as BF
from bench_fozerax import _lens, _rnd, _state
from bench_sipazen import VOCAB, _cu, _line, _median_ms, _tables, family_throughput

CHUNK, CAP = 1024, 20.0
SFU_PER_SM_CLOCK = 16


def subivik_config(s, **over):
    W = s["width"]
    par = {"type": "parallel",
           "mixer": {"left": {"heads": s["heads"], "kv_heads": s["kv"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": CAP},
                     "right": {"heads": W // 64, "dim": 64}, "left_scale": 0.7, "right_scale": 0.7}}
    att = {"heads": s["heads"], "kv_heads": s["kv"], "dim": 64, "vdim": 128, "scale": 64 ** -0.5, "diff": 0.5, "mask": {"size": CHUNK}}
    mlp = {"kind": "moe", "router": {"experts": s["experts"], "top": s["top"], "scale": 2.0}, "expert": {"ff": s["ff"]}}
    layers = [par, {"type": "attention", "mixer": att}, par, {"type": "attention", "mixer": {**att, "kv_from": 1}}]
    return {"architecture": "Subivik", "vocab": VOCAB, "width": W, "norm": {"eps": 1e-6}, "layers": [{**l, "mlp": mlp} for l in layers], **over}


def fozerax_config(s):
    c = BF.fozerax_config(s)
    for l in c["layers"]:
        l["mlp"] = {k: v for k, v in l["mlp"].items() if k != "shared"}
    return c


# ------------------------------------------------------------------------------------------------- kernels
def _wave(dev):
    from minivllm_b200 import synth
    lens = [int(n) for n in synth.prefill_inputs(num_seqs=32, len_lo=128, len_hi=2048)["lens"]]
    return lens, sum(lens), _cu(lens, dev)


def _sfu(d, weights, per_weight):
    """Fraction of the special-function unit's rate, at the SM clock's maximum, that the given weights take up."""
    d["frac_sfu"] = weights * per_weight / (d["us"] * 1e-6) / (148 * SFU_PER_SM_CLOCK * 1965e6)
    return d


def _rates(dev, heads):
    return torch.rand(heads, device=dev), torch.rand(heads, device=dev), torch.randn(heads, heads, device=dev) * heads ** -0.5


def kernel_talk_prefill(dev, pk, iters=20, heads=16, kv=4, dim=128, vdim=128):
    """The weights of every head over the values of every value head; FLOPs: those of the plain attention (frac_bf16) and
    those of the products that are made (frac_bf16_made)."""
    from minivllm_b200.layers import talk_attention as TA
    lens, T, cu = _wave(dev)
    q, k, v, (r1, r2, _) = _rnd(dev, T, heads * dim), _rnd(dev, T, kv * dim), _rnd(dev, T, kv * vdim), _rates(dev, heads)
    ms = _median_ms(lambda: TA.talk_prefill(q, k, v, cu, cu, kv, dim, vdim, dim ** -0.5, r1, r2, CAP), iters)
    pairs = sum(n * (n + 1) // 2 for n in lens)
    d = _line(ms, pk, flops=2.0 * heads * (dim + vdim) * pairs, nbytes=2 * T * (heads * dim + kv * (dim + vdim) + heads * kv * vdim))
    passes = -(-kv // (4 // (vdim // 64)))
    d["frac_bf16_made"] = 2.0 * heads * (passes * dim + kv * vdim) * pairs / ms / 1e9 / pk["bf16_tflops"]
    return _sfu(d, passes * heads * pairs, 1.875)


def kernel_head_mix(dev, pk, iters=20, rows=16384, heads=16, kv=4, vdim=128):
    from minivllm_b200.layers import talk_attention as TA
    a, talk, out = _rnd(dev, rows, heads, kv, vdim), _rates(dev, heads)[2], _rnd(dev, rows, heads * vdim)
    ms = _median_ms(lambda: TA.head_mix(a, talk, out, 0.7), iters)
    return _line(ms, pk, nbytes=(a.numel() + out.numel()) * 2)


def kernel_talk_decode(dev, pk, iters=20, batch=64, heads=16, kv=4, dim=128, vdim=128):
    from minivllm_b200.layers import talk_attention as TA
    ctx = torch.randint(512, 1537, (batch,), generator=torch.Generator().manual_seed(0)).tolist()
    tables, blocks = _tables(batch, ctx, 64, dev)
    cache, q, (r1, r2, talk) = _rnd(dev, blocks, 64, kv * (dim + vdim)), _rnd(dev, batch, heads * dim), _rates(dev, heads)
    pos, out = torch.tensor(ctx, device=dev, dtype=torch.int64) - 1, _rnd(dev, batch, heads * vdim)
    ms = _median_ms(lambda: TA.talk_decode(q, cache, tables, pos, kv, dim, vdim, dim ** -0.5, r1, r2, CAP, talk, out), iters)
    return _line(ms, pk, nbytes=sum(ctx) * kv * (dim + vdim) * 2 + batch * heads * (dim + vdim) * 2)


def _diff(dev, rows, heads, kv, dim, vdim):
    return _rnd(dev, rows, heads * 2 * dim), _rnd(dev, rows, heads * vdim), torch.empty(rows, heads * vdim, dtype=torch.bfloat16, device=dev)


def kernel_diff_prefill(dev, pk, iters=20, heads=16, kv=4, dim=64, vdim=128, chunk=CHUNK):
    """Two maps of 64 against the like kernel's one of 128; both maps meet the values."""
    from minivllm_b200.layers import diff_attention as DA
    lens, T, cu = _wave(dev)
    (q, gate, out), rows = _diff(dev, T, heads, kv, dim, vdim), _rnd(dev, T, kv * (2 * dim + vdim))
    ms = _median_ms(lambda: DA.diff_prefill(q, rows, cu, cu, chunk, gate, 0.4, 0.5, 1e-6, heads, kv, dim, vdim, dim ** -0.5, out), iters)
    pairs = sum(i % chunk + 1 for n in lens for i in range(n))
    return _sfu(_line(ms, pk, flops=4.0 * heads * (dim + vdim) * pairs,
                      nbytes=2 * T * (heads * (2 * dim + 2 * vdim) + kv * (2 * dim + vdim))), 2 * heads * pairs, 1)


def kernel_diff_decode(dev, pk, iters=20, batch=64, heads=16, kv=4, dim=64, vdim=128, chunk=CHUNK):
    from minivllm_b200.layers import diff_attention as DA
    ctx = (chunk + torch.randint(chunk // 2, chunk, (batch,), generator=torch.Generator().manual_seed(0))).tolist()
    tables, blocks = _tables(batch, ctx, 64, dev)
    cache, (q, gate, out) = _rnd(dev, blocks, 64, kv * (2 * dim + vdim)), _diff(dev, batch, heads, kv, dim, vdim)
    pos = torch.tensor(ctx, device=dev, dtype=torch.int64) - 1
    ms = _median_ms(lambda: DA.diff_decode(q, cache, tables, pos, chunk, gate, 0.4, 0.5, 1e-6, heads, kv, dim, vdim, dim ** -0.5, out), iters)
    return _line(ms, pk, nbytes=sum((c - 1) % chunk + 1 for c in ctx) * kv * (2 * dim + vdim) * 2 + batch * heads * (2 * dim + 2 * vdim) * 2)


def kernel_norm_store(dev, pk, iters=20, rows=16384, heads=16, kv=4, dim=64, vdim=128):
    from minivllm_b200.layers.rotary_attention import qkv_rope_store
    qn, kn, vn = heads * 2 * dim, kv * 2 * dim, kv * vdim
    p, w = _rnd(dev, rows, qn + kn + vn), _rnd(dev, dim)
    cache, slots = _rnd(dev, rows // 64, 64, kn + vn), torch.arange(rows, device=dev)
    ms = _median_ms(lambda: qkv_rope_store(p[:, :qn], p[:, qn:qn + kn], p[:, qn + kn:], w, w, None, 1e-6, slots, None, 0, None, 2 * heads,
                                           2 * kv, cache, slots, packed=True, v_heads=kv), iters)
    return _line(ms, pk, nbytes=rows * (2 * qn + 3 * (kn + vn)) * 2)


def _time(dev, tokens, heads, K):
    n = heads * K
    return _rnd(dev, 4, tokens, n).unbind(0), torch.randn(tokens, n, device=dev) - 3, _rnd(dev, n), _rnd(dev, heads, K)


def kernel_time_scan(dev, pk, iters=20, seqs=16, tokens=16384, heads=32, K=64):
    from minivllm_b200.layers import time_mix as L
    m, ((r, k, v, _), z, w0, u) = _state(dev, seqs, heads, K, K), _time(dev, tokens, heads, K)
    cu = _cu(_lens(seqs, tokens), dev)
    ms = _median_ms(lambda: L.time_scan(r, k, v, z, w0, u, cu, m["slots"], m["starts"], m["S"], heads, K, K), iters)
    return _line(ms, pk, nbytes=tokens * heads * K * 12 + m["S"].numel() * 8)


def kernel_time_step(dev, pk, iters=20, batch=64, heads=32, K=64):
    from minivllm_b200.layers import time_mix as L
    m, ((r, k, v, g), z, w0, u) = _state(dev, batch, heads, K, K), _time(dev, batch, heads, K)
    ms = _median_ms(lambda: L.time_scan(r, k, v, z, w0, u, None, m["slots"], m["starts"], m["S"], heads, K, K, gate=g, norm_w=w0, eps=1e-6), iters)
    return _line(ms, pk, nbytes=m["S"].numel() * 8 + batch * heads * K * 14)


def kernel_tanh_step(dev, pk, iters=20, rows=16384, width=2048, mixes=0, seqs=16, top=0):
    from minivllm_b200.layers import tanh_norm as TN
    from minivllm_b200.utils.context import reset_context, set_context
    x, y, w = torch.zeros(rows, width, device=dev), _rnd(dev, rows * max(top, 1), width), _rnd(dev, width)
    if top:
        y = (y, torch.randperm(rows * top, device=dev).to(torch.int32).view(rows, top), torch.rand(rows, top, device=dev))
    shift, cu = None, _cu(_lens(seqs, rows), dev)
    if mixes:
        shift = TN.TokenShift(torch.rand(mixes, width, device=dev).bfloat16())
        shift.slot_state = {"h": _rnd(dev, seqs, width)}
    set_context(True, cu, portion_cu_q=cu, num_decode=0, state_slots=torch.arange(seqs, dtype=torch.int32, device=dev),
                state_starts=torch.ones(seqs, dtype=torch.int32, device=dev))
    entry = TN.TanhEntry(torch.tensor(0.7), w, w, shift)
    ms = _median_ms(lambda: TN.tanh_step(x, y, entry), iters)
    reset_context()
    return _line(ms, pk, nbytes=rows * width * (10 + 2 * max(top, 1) + 2 * mixes))


def kernel_xielu(dev, pk, iters=20, rows=16384, cols=4096):
    from minivllm_b200.layers.mlp import xielu
    z = _rnd(dev, rows, cols)
    return _line(_median_ms(lambda: xielu(z, 0.7, 1.2), iters), pk, nbytes=rows * cols * 4)


def kernel_route(dev, pk, iters=20, tokens=16384, experts=64, top=6):
    from minivllm_b200.layers import moe
    z = torch.randn(tokens, experts, device=dev)
    return _line(_median_ms(lambda: moe.route(z, None, top, over_all=True, scale=2.0), iters), pk, nbytes=tokens * (experts + 2 * top) * 4)


def kernel_head_norm(dev, pk, iters=20, rows=16384, heads=32, dim=64):
    from minivllm_b200.layers import group_norm as GN
    y, z, w = _rnd(dev, rows, heads * dim), _rnd(dev, rows, heads * dim), _rnd(dev, heads * dim)
    out = _rnd(dev, rows, 2 * heads * dim)[:, heads * dim:]
    ms = _median_ms(lambda: GN.head_norm_gate(y, z, w, heads, 1e-6, out=out, mult=0.7), iters)
    return _line(ms, pk, nbytes=rows * heads * dim * 6)


# kernel -> (what runs it, the like kernel of Fozerax in bench_fozerax.KERNELS)
KERNELS = {
    "talk_prefill_32seq_16heads": (kernel_talk_prefill, "window_prefill_32seq_16heads"),
    "head_mix_16384x16x4x128": (kernel_head_mix, "pair_residual_norm_16384x2048"),
    "talk_decode_b64_16heads": (kernel_talk_decode, "window_decode_b64_16heads"),
    "diff_prefill_32seq_16heads": (kernel_diff_prefill, "window_prefill_32seq_16heads"),
    "diff_decode_b64_16heads": (kernel_diff_decode, "window_decode_b64_16heads"),
    "qk_norm_store_16384tok": (kernel_norm_store, "kv_norm_store_16384tok"),
    "time_scan_16x1024tok": (kernel_time_scan, "gla_scan_16x1024tok"),
    "time_scan_1x16384tok": (lambda d, p, iters=20: kernel_time_scan(d, p, iters, seqs=1), "gla_scan_1x16384tok"),
    "time_step_b64": (kernel_time_step, "gla_step_b64"),
    "tanh_step_16384x2048": (kernel_tanh_step, "post_residual_norm_16384x2048"),
    "tanh_step_5_mixtures_16384x2048": (lambda d, p, iters=20: kernel_tanh_step(d, p, iters, mixes=5), "post_residual_norm_16384x2048"),
    "tanh_step_experts_16384x2048": (lambda d, p, iters=20: kernel_tanh_step(d, p, iters, top=6), "moe_residual_norm_16384x2048"),
    "xielu_16384x4096": (kernel_xielu, "gelu_glu_16384x4096"),
    "route_over_all_16384tok": (kernel_route, "route_in_groups_16384tok"),
    "head_norm_gate_16384x2048": (kernel_head_norm, "head_norm_gate_16384x2048"),
}


def run(device, pk, steps, only=None):
    from minivllm_b200.layers.attention import prefill_error_code
    kernels, like = {}, {}
    frac = lambda d: max(d.get("frac_hbm", 0.0), d.get("frac_bf16", 0.0))
    for name, (fn, other) in KERNELS.items():
        if only and only != name:
            continue
        kernels[name] = fn(device, pk, iters=max(5, steps))
        if other not in like:
            like[other] = BF.KERNELS[other][0](device, pk, iters=max(5, steps))
        torch.cuda.empty_cache()
        kernels[name].update(like=other, like_us=like[other]["us"], like_frac=frac(like[other]),
                             frac_over_like=frac(kernels[name]) / frac(like[other]))
    sizes = {}
    if not only:
        for name, s in BF.SIZES.items():
            sizes[name] = {"subivik": family_throughput(subivik_config(s)), "fozerax": family_throughput(fozerax_config(s))}
    head = sizes.get("w2048", {}).get("subivik", {})
    return {"metric": "Subivik prefill tokens/s, width 2048, 4 layers, one wave of 16 x 1024 tokens",
            "value": head.get("prefill_tok_s"), "unit": "tok/s", "n_gpus": 1, "steps": steps, "warmup": 3,
            "higher_is_better": True, "data": "synthetic", "dtype": "bf16",
            "config": {"workload": "subivik family beside the fozerax family at equal size; kernels at the shapes of width 2048"},
            "extra": {"throughput": sizes, "kernels": kernels, "error_word": prefill_error_code(device)}}
