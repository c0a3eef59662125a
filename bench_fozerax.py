"""`bench.py --workload fozerax`: throughput of the Fozerax family beside the Sipazen family (the closest one: recurrent
layers, mixtures of experts) at equal size, and every kernel of the family against its roofline, beside the like kernel of
Sipazen.

Sizes: random weights, four layers (windowed attention beside a gated delta rule, and gated linear attention, in turn),
experts of a mid-size mixture; the Sipazen model of a size has the same width, layer count, vocabulary and experts.
Prefill is one wave of 16 prompts x 1,024 tokens, decode the captured graph with 64 sequences behind 1,024-token contexts;
both timed on the device with CUDA events around the engine's own step, per-step inputs of more than the L2 size (weights,
cache and state).
"""
import torch

import bench_sipazen as BS
from bench_sipazen import VOCAB, _cu, _line, _median_ms, _tables, family_throughput, sipazen_config

SIZES = {
    "w1024": dict(width=1024, heads=8, kv=2, rheads=8, rkv=4, gheads=4, gdim=128, gvdim=256, experts=32, top=4, ff=512, shared=1024),
    "w2048": dict(width=2048, heads=16, kv=4, rheads=16, rkv=8, gheads=8, gdim=128, gvdim=256, experts=64, top=6, ff=1024, shared=2048),
    "w4096": dict(width=4096, heads=32, kv=8, rheads=32, rkv=16, gheads=16, gdim=128, gvdim=256, experts=64, top=6, ff=1536, shared=3072),
}
WINDOW, BIAS_MAX = 1024, 128


def fozerax_config(s, **over):
    par = {"type": "parallel",
           "mixer": {"left": {"heads": s["heads"], "kv_heads": s["kv"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                              "bias_max": BIAS_MAX, "mask": {"size": WINDOW}},
                     "right": {"heads": s["rheads"], "kv_heads": s["rkv"], "dim": 128, "vdim": 128, "conv": 4}}}
    gla = {"type": "gla", "mixer": {"heads": s["gheads"], "dim": s["gdim"], "vdim": s["gvdim"], "tau": 16.0}}
    mlp = {"kind": "moe", "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": 8, "keep": 4}},
           "expert": {"ff": s["ff"], "limit": 7.0}, "shared": {"ff": s["shared"], "limit": 7.0}}
    c = {"architecture": "Fozerax", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-6},
         "layers": [{**l, "mlp": mlp} for l in (par, gla, par, gla)]}
    return {**c, **over}


# ------------------------------------------------------------------------------------------------- kernels
def _rnd(dev, *shape):
    return torch.randn(*shape, device=dev, dtype=torch.float32).to(torch.bfloat16)


def _bias(dev, heads, window):
    from minivllm_b200.layers import window_attention as WA
    return WA.distance_bias(_rnd(dev, 32, heads), BIAS_MAX, window)


def kernel_window_prefill(dev, pk, iters=20, heads=16, kv=4, dim=128, vdim=128, window=WINDOW):
    from minivllm_b200 import synth
    from minivllm_b200.layers import window_attention as WA
    lens = [int(n) for n in synth.prefill_inputs(num_seqs=32, len_lo=128, len_hi=2048)["lens"]]
    T, cu = sum(lens), _cu(lens, dev)
    q, rows, bias, sink = _rnd(dev, T, heads * dim), _rnd(dev, T, kv * (dim + vdim)), _bias(dev, heads, window), _rnd(dev, heads)
    ms = _median_ms(lambda: WA.window_prefill(q, rows, cu, cu, kv, dim, vdim, window, dim ** -0.5, bias, sink), iters)
    pairs = sum(min(i + 1, window) for n in lens for i in range(n))
    return _line(ms, pk, flops=2.0 * heads * (dim + vdim) * pairs,
                 nbytes=2 * T * (heads * (dim + vdim) + kv * (dim + vdim)))


def kernel_window_decode(dev, pk, iters=20, batch=64, heads=16, kv=4, dim=128, vdim=128, window=WINDOW):
    from minivllm_b200.layers import window_attention as WA
    g = torch.Generator().manual_seed(0)
    ctx = torch.randint(1024, 4097, (batch,), generator=g).tolist()
    tables, blocks = _tables(batch, ctx, 64, dev)
    cache, q = _rnd(dev, blocks, 64, kv * (dim + vdim)), _rnd(dev, batch, heads * dim)
    pos, bias, sink = torch.tensor(ctx, device=dev, dtype=torch.int64) - 1, _bias(dev, heads, window), _rnd(dev, heads)
    ms = _median_ms(lambda: WA.window_decode(q, cache, tables, pos, kv, dim, vdim, window, dim ** -0.5, bias, sink), iters)
    return _line(ms, pk, nbytes=sum(min(c, window) for c in ctx) * kv * (dim + vdim) * 2 + batch * heads * (dim + vdim) * 2)


def kernel_norm_store(dev, pk, iters=20, rows=16384, qn=2048, kn=512, vn=512):
    from minivllm_b200.layers import window_attention as WA
    p, wq, wk = _rnd(dev, rows, qn + kn + vn), _rnd(dev, qn), _rnd(dev, kn)
    cache, slots = _rnd(dev, rows // 64, 64, kn + vn), torch.arange(rows, device=dev)
    ms = _median_ms(lambda: WA.kv_norm_store(p[:, :qn], p[:, qn:qn + kn], p[:, qn + kn:], wq, wk, 1e-6, cache, slots, packed=True), iters)
    return _line(ms, pk, nbytes=rows * (2 * qn + 3 * (kn + vn)) * 2)


def _lens(seqs, tokens):
    return [tokens // seqs] * seqs


def _state(dev, seqs, heads, K, V):
    return dict(slots=torch.arange(seqs, dtype=torch.int32, device=dev), starts=torch.ones(seqs, dtype=torch.int32, device=dev),
                S=torch.zeros(seqs, heads, K, V, device=dev))


def kernel_gla_scan(dev, pk, iters=20, seqs=16, tokens=16384, heads=8, K=128, V=256):
    from minivllm_b200.layers import gla as L
    m, p, z = _state(dev, seqs, heads, K, V), _rnd(dev, tokens, 2 * heads * K + heads * V), _rnd(dev, tokens, heads * K) + 3
    q, k, v = p.split([heads * K, heads * K, heads * V], 1)
    cu = _cu(_lens(seqs, tokens), dev)
    ms = _median_ms(lambda: L.gla_scan(q, k, v, z, 16.0, cu, m["slots"], m["starts"], m["S"], heads, K, V), iters)
    return _line(ms, pk, nbytes=tokens * heads * (3 * K + 2 * V) * 2 + m["S"].numel() * 8)


def kernel_gla_step(dev, pk, iters=20, batch=64, heads=8, K=128, V=256):
    from minivllm_b200.layers import gla as L
    m, p, z = _state(dev, batch, heads, K, V), _rnd(dev, batch, 2 * heads * K + 2 * heads * V), _rnd(dev, batch, heads * K) + 3
    q, k, v, g = p.split([heads * K, heads * K, heads * V, heads * V], 1)
    w = _rnd(dev, V)
    ms = _median_ms(lambda: L.gla_scan(q, k, v, z, 16.0, None, m["slots"], m["starts"], m["S"], heads, K, V, gate=g, norm_w=w, eps=1e-6), iters)
    return _line(ms, pk, nbytes=m["S"].numel() * 8 + batch * heads * (3 * K + 3 * V) * 2)


def _delta(dev, tokens, heads, kv, K, V):
    ch = 2 * kv * K + heads * V
    return dict(u=_rnd(dev, tokens, ch), ba=_rnd(dev, tokens, 2 * heads), A_log=_rnd(dev, heads), dt=_rnd(dev, heads) - 2, ch=ch,
                g=_rnd(dev, tokens, heads * V), w=_rnd(dev, V), cw=_rnd(dev, ch, 4))


def kernel_delta_scan(dev, pk, iters=20, seqs=16, tokens=16384, heads=16, kv=8, K=128, V=128):
    from minivllm_b200.layers import gated_delta as L
    m, d, cu = _state(dev, seqs, heads, K, V), _delta(dev, tokens, heads, kv, K, V), _cu(_lens(seqs, tokens), dev)
    ms = _median_ms(lambda: L.delta_scan(d["u"], d["ba"][:, :heads], d["ba"][:, heads:], d["A_log"], d["dt"], cu, m["slots"], m["starts"],
                                         m["S"], heads, kv, K, V), iters)
    return _line(ms, pk, nbytes=tokens * (d["ch"] + heads * V + 2 * heads) * 2 + m["S"].numel() * 8)


def kernel_delta_step(dev, pk, iters=20, batch=64, heads=16, kv=8, K=128, V=128):
    from minivllm_b200.layers import gated_delta as L
    m, d = _state(dev, batch, heads, K, V), _delta(dev, batch, heads, kv, K, V)
    conv = _rnd(dev, batch, 3, d["ch"])
    ms = _median_ms(lambda: L.delta_scan(d["u"], d["ba"][:, :heads], d["ba"][:, heads:], d["A_log"], d["dt"], None, m["slots"], m["starts"],
                                         m["S"], heads, kv, K, V, conv_w=d["cw"], conv_state=conv, gate=d["g"], norm_w=d["w"], eps=1e-6), iters)
    return _line(ms, pk, nbytes=m["S"].numel() * 8 + batch * (4 * d["ch"] + 2 * heads * V) * 2)


def kernel_conv(dev, pk, iters=20, seqs=16, tokens=16384, heads=16, kv=8, K=128, V=128):
    from minivllm_b200.layers.short_conv import conv_silu
    m, d, cu = _state(dev, seqs, 1, 1, 1), _delta(dev, tokens, heads, kv, K, V), _cu(_lens(seqs, tokens), dev)
    conv = _rnd(dev, seqs, 3, d["ch"])
    ms = _median_ms(lambda: conv_silu(d["u"], d["cw"], None, cu, m["slots"], m["starts"], conv), iters)
    return _line(ms, pk, nbytes=tokens * d["ch"] * 4)


def kernel_pair_norm(dev, pk, iters=20, rows=16384, width=2048):
    from minivllm_b200.layers import group_norm as GN
    x, a, b = torch.zeros(rows, width, device=dev), _rnd(dev, rows, width), _rnd(dev, rows, width)
    w = [_rnd(dev, width) for _ in range(3)]
    ms = _median_ms(lambda: GN.pair_residual_norm(x, a, w[0], b, w[1], w[2], None, 1.0, 1, 1e-6), iters)
    return _line(ms, pk, nbytes=rows * width * 14)


def kernel_post_norm(dev, pk, iters=20, rows=16384, width=2048):
    from minivllm_b200.layers import group_norm as GN
    x, y, w = torch.zeros(rows, width, device=dev), _rnd(dev, rows, width), _rnd(dev, width)
    ms = _median_ms(lambda: GN.gated_residual_norm(x, y, None, None, w, None, 1.0, 1, 1e-6), iters)
    return _line(ms, pk, nbytes=rows * width * 12)


def kernel_moe_residual(dev, pk, iters=20, rows=16384, width=2048, top=6):
    from minivllm_b200.layers import group_norm as GN
    from minivllm_b200.layers import moe
    x, y, w, sh = torch.zeros(rows, width, device=dev), _rnd(dev, rows * top, width), _rnd(dev, width), _rnd(dev, rows, width)
    idx, tw = moe.route(torch.randn(rows, 64, device=dev), None, top)
    pos, _, _ = moe.sort_by_expert(idx, 64)
    ms = _median_ms(lambda: GN.moe_residual_norm(x, y, pos, tw, sh, None, None, None, w, None, 1.0, 1, 1e-6), iters)
    return _line(ms, pk, nbytes=rows * width * (12 + 2 * top))


def kernel_head_norm(dev, pk, iters=20, rows=16384, heads=16, vdim=128):
    from minivllm_b200.layers import group_norm as GN
    y, z, w = _rnd(dev, rows, heads * vdim), _rnd(dev, rows, heads * vdim), _rnd(dev, vdim)
    ms = _median_ms(lambda: GN.head_norm_gate(y, z, w, heads, 1e-6), iters)
    return _line(ms, pk, nbytes=rows * heads * vdim * 6)


def kernel_glu(dev, pk, iters=20, rows=16384, cols=4096, act="gelu_tanh"):
    from minivllm_b200.layers import group_norm as GN
    p = _rnd(dev, rows, 2 * cols)
    ms = _median_ms(lambda: GN.gate_mul(p[:, cols:], p[:, :cols], act, limit=7.0), iters)
    return _line(ms, pk, nbytes=rows * cols * 6)


def kernel_route(dev, pk, iters=20, tokens=16384, experts=64, top=6):
    from minivllm_b200.layers import moe
    z = torch.randn(tokens, experts, device=dev)
    return _line(_median_ms(lambda: moe.route(z, None, top, 8, 4), iters), pk, nbytes=tokens * (experts + 2 * top) * 4)


def kernel_grouped(dev, pk, tokens, iters=20, experts=64, top=6, width=2048, ff=1024):
    from minivllm_b200.layers import moe
    idx, _ = moe.route(torch.randn(tokens, experts, device=dev), None, top)
    _, _, offsets = moe.sort_by_expert(idx, experts)
    used = int((offsets[1:] > offsets[:-1]).sum())
    x, w = _rnd(dev, tokens * top, width), _rnd(dev, experts, 2 * ff, width)
    ms = _median_ms(lambda: moe.grouped_linear(x, w, offsets, True, act="clamped", limit=7.0), iters)
    return _line(ms, pk, nbytes=used * 2 * ff * width * 2 + (x.numel() + tokens * top * ff) * 2, flops=2.0 * tokens * top * 2 * ff * width)


# kernel -> (what runs it, the like kernel of Sipazen in bench_sipazen.KERNELS)
KERNELS = {
    "window_prefill_32seq_16heads": (kernel_window_prefill, "latent_prefill_32seq_16heads"),
    "window_decode_b64_16heads": (kernel_window_decode, "latent_decode_b64_16heads"),
    "kv_norm_store_16384tok": (kernel_norm_store, "latent_prep_16384tok"),
    "gla_scan_16x1024tok": (kernel_gla_scan, "ssm_chunk_scan_16x1024tok"),
    "gla_scan_1x16384tok": (lambda d, p, iters=20: kernel_gla_scan(d, p, iters, seqs=1), "ssm_chunk_scan_1x16384tok"),
    "gla_step_b64": (kernel_gla_step, "ssm_step_b64"),
    "delta_scan_16x1024tok": (kernel_delta_scan, "ssm_chunk_scan_16x1024tok"),
    "delta_scan_1x16384tok": (lambda d, p, iters=20: kernel_delta_scan(d, p, iters, seqs=1), "ssm_chunk_scan_1x16384tok"),
    "delta_step_b64": (kernel_delta_step, "ssm_step_b64"),
    "conv_silu_16384tok": (kernel_conv, "conv_silu_16384tok"),
    "pair_residual_norm_16384x2048": (kernel_pair_norm, "gated_residual_norm_16384x2048"),
    "post_residual_norm_16384x2048": (kernel_post_norm, "gated_residual_norm_16384x2048"),
    "moe_residual_norm_16384x2048": (kernel_moe_residual, "moe_residual_norm_16384x2048"),
    "head_norm_gate_16384x2048": (kernel_head_norm, "gated_group_norm_16384x4096"),
    "gelu_glu_16384x4096": (kernel_glu, "gate_mul_16384x2048"),
    "clamped_glu_16384x4096": (lambda d, p, iters=20: kernel_glu(d, p, iters, act="clamped"), "gate_mul_16384x2048"),
    "route_in_groups_16384tok": (kernel_route, None),
    "grouped_gate_up_16384tok": (lambda d, p, iters=20: kernel_grouped(d, p, 16384, iters), "grouped_gate_up_16384tok"),
    "grouped_gate_up_64tok": (lambda d, p, iters=20: kernel_grouped(d, p, 64, iters), "grouped_gate_up_64tok"),
}


def run(device, pk, steps, only=None):
    from minivllm_b200.layers.attention import prefill_error_code
    kernels, like = {}, {}
    for name, (fn, other) in KERNELS.items():
        if only and only != name:
            continue
        kernels[name] = fn(device, pk, iters=max(5, steps))
        if other and other not in like:
            like[other] = BS.KERNELS[other](device, pk, iters=max(5, steps))
        torch.cuda.empty_cache()
        if other:
            frac = lambda d: max(d.get("frac_hbm", 0.0), d.get("frac_bf16", 0.0))
            kernels[name].update(like=other, like_frac=frac(like[other]), frac_over_like=frac(kernels[name]) / frac(like[other]))
    sizes = {}
    if not only:
        for name, s in SIZES.items():
            sizes[name] = {"fozerax": family_throughput(fozerax_config(s)), "sipazen": family_throughput(sipazen_config(BS.SIZES[name]))}
    head = sizes.get("w2048", {}).get("fozerax", {})
    return {"metric": "Fozerax prefill tokens/s, width 2048, 4 layers, one wave of 16 x 1024 tokens",
            "value": head.get("prefill_tok_s"), "unit": "tok/s", "n_gpus": 1, "steps": steps, "warmup": 3,
            "higher_is_better": True, "data": "synthetic", "dtype": "bf16",
            "config": {"workload": "fozerax family beside the sipazen family at equal size; kernels at the shapes of width 2048"},
            "extra": {"throughput": sizes, "kernels": kernels, "error_word": prefill_error_code(device)}}
