"""`bench.py --workload dafotar`: throughput of the Dafotar family beside the Fozerax family (the closest one: windowed
attention and recurrences on a matrix state) at equal size, and every kernel of the family against its roofline, beside the
like kernel of Fozerax.

Sizes: random weights, four layers (windowed attention and matrix memory in turn, the second attention on the first one's
keys and values), two residual streams, dense feed-forwards; the Fozerax model of a size has the same width, layer count,
vocabulary, heads and feed-forwards.  Prefill is one wave of 16 prompts x 1,024 tokens, decode the captured graph with 64
sequences behind 1,024-token contexts; both timed on the device with CUDA events around the engine's own step, per-step
inputs of more than the L2 size (weights, cache and state).
"""
import torch

import bench_fozerax as BF
from bench_fozerax import WINDOW, _lens, _rnd, _state
from bench_sipazen import VOCAB, _cu, _line, _median_ms, _tables, family_throughput

SIZES = {"w1024": 1024, "w2048": 2048, "w4096": 4096}


def dafotar_config(name, **over):
    s, W = BF.SIZES[name], SIZES[name]
    att = {"heads": s["heads"], "kv_heads": s["kv"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": WINDOW},
           "rot": {"base": 1e5, "dims": 128}}
    mem = {"type": "mlstm", "mixer": {"heads": s["gheads"], "dim": s["gdim"], "vdim": s["gvdim"], "gate_cap": 15.0}}
    layers = [{"type": "attention", "mixer": att}, mem, {"type": "attention", "mixer": {**att, "kv_from": 0}}, mem]
    return {"architecture": "Dafotar", "vocab": VOCAB, "width": W, "streams": 2, "canon": {"taps": 4}, "norm": {"eps": 1e-6},
            "layers": [{**l, "mlp": {"kind": "dense", "ff": 3 * W}} for l in layers], **over}


def fozerax_config(name):
    c = BF.fozerax_config(BF.SIZES[name])
    return {**c, "layers": [{**l, "mlp": {"kind": "dense", "ff": 3 * SIZES[name]}} for l in c["layers"]]}


# ------------------------------------------------------------------------------------------------- kernels
def _turn(dev, vdim, rows=4096):
    from minivllm_b200.layers.rotary_attention import turn_table
    return turn_table(1e5, vdim, rows, dev)


def kernel_window_prefill(dev, pk, iters=20, heads=16, kv=4, dim=128, vdim=128, window=WINDOW):
    from minivllm_b200 import synth
    from minivllm_b200.layers import window_attention as WA
    lens = [int(n) for n in synth.prefill_inputs(num_seqs=32, len_lo=128, len_hi=2048)["lens"]]
    T, cu = sum(lens), _cu(lens, dev)
    q, rows, pos = _rnd(dev, T, heads * dim), _rnd(dev, T, kv * (dim + vdim)), torch.cat([torch.arange(n) for n in lens]).to(dev)
    turn = _turn(dev, vdim)
    ms = _median_ms(lambda: WA.window_prefill(q, rows, cu, cu, kv, dim, vdim, window, dim ** -0.5, turn=turn, positions=pos), iters)
    pairs = sum(min(i + 1, window) for n in lens for i in range(n))
    return _line(ms, pk, flops=2.0 * heads * (dim + vdim) * pairs,
                 nbytes=2 * T * (heads * (dim + vdim) + kv * (dim + vdim)))


def kernel_window_decode(dev, pk, iters=20, batch=64, heads=16, kv=4, dim=128, vdim=128, window=WINDOW):
    from minivllm_b200.layers import window_attention as WA
    ctx = torch.randint(1024, 4097, (batch,), generator=torch.Generator().manual_seed(0)).tolist()
    tables, blocks = _tables(batch, ctx, 64, dev)
    cache, q = _rnd(dev, blocks, 64, kv * (dim + vdim)), _rnd(dev, batch, heads * dim)
    pos, turn = torch.tensor(ctx, device=dev, dtype=torch.int64) - 1, _turn(dev, vdim)
    ms = _median_ms(lambda: WA.window_decode(q, cache, tables, pos, kv, dim, vdim, window, dim ** -0.5, turn=turn), iters)
    return _line(ms, pk, nbytes=sum(min(c, window) for c in ctx) * kv * (dim + vdim) * 2 + batch * heads * (dim + vdim) * 2)


def kernel_rope_store(dev, pk, iters=20, rows=16384, heads=16, kv=4, dim=128, vdim=128):
    from minivllm_b200.layers import rotary_attention as RA
    from minivllm_b200.layers.latent_attention import rope_table
    qn, kn, vn = heads * dim, kv * dim, kv * vdim
    p, w, temp = _rnd(dev, rows, qn + kn + vn), _rnd(dev, dim), _rnd(dev, heads)
    cache, slots, pos = _rnd(dev, rows // 64, 64, kn + vn), torch.arange(rows, device=dev), torch.arange(rows, device=dev) % 1024
    table = rope_table(1e5, dim, 4096, dev)
    ms = _median_ms(lambda: RA.qkv_rope_store(p[:, :qn], p[:, qn:qn + kn], p[:, qn + kn:], w, w, temp, 1e-6, pos, table, dim, table,
                                              heads, kv, cache, slots, packed=True), iters)
    return _line(ms, pk, nbytes=rows * (2 * qn + 3 * (kn + vn)) * 2)


def _memory(dev, tokens, heads, K, V, gate=False):
    sizes = [heads * K, heads * K, heads * V] + ([heads * V] if gate else [])
    z = torch.randn(tokens, 2 * heads, device=dev)
    z[:, heads:] += 4
    return _rnd(dev, tokens, sum(sizes)).split(sizes, 1), z, _rnd(dev, heads)


def kernel_mlstm_scan(dev, pk, iters=20, seqs=16, tokens=16384, heads=8, K=128, V=256):
    """All launches of a portion's recurrence, the chain of maxima among them."""
    from minivllm_b200.layers import mlstm as L
    m, ((q, k, v), z, b) = _state(dev, seqs, heads, K, V), _memory(dev, tokens, heads, K, V)
    n, mx, cu = torch.zeros(seqs, heads, K, device=dev), torch.zeros(seqs, heads, device=dev), _cu(_lens(seqs, tokens), dev)

    def run():
        chain = L.mlstm_gates(z, b, b, 15.0, cu, m["slots"], m["starts"], mx, heads)
        L.mlstm_scan(q, k, v, chain, cu, m["slots"], m["starts"], m["S"], n, heads, K, V)
    return _line(_median_ms(run, iters), pk, nbytes=tokens * heads * ((2 * K + 2 * V) * 2 + 12) + m["S"].numel() * 8)


def kernel_mlstm_gates(dev, pk, iters=20, seqs=16, tokens=16384, heads=8):
    from minivllm_b200.layers import mlstm as L
    m, (_, z, b) = _state(dev, seqs, heads, 1, 1), _memory(dev, tokens, heads, 1, 1)
    mx, cu = torch.zeros(seqs, heads, device=dev), _cu(_lens(seqs, tokens), dev)
    ms = _median_ms(lambda: L.mlstm_gates(z, b, b, 15.0, cu, m["slots"], m["starts"], mx, heads), iters)
    return _line(ms, pk, nbytes=tokens * heads * 24)


def kernel_mlstm_step(dev, pk, iters=20, batch=64, heads=8, K=128, V=256):
    from minivllm_b200.layers import mlstm as L
    m, ((q, k, v, g), _, b) = _state(dev, batch, heads, K, V), _memory(dev, batch, heads, K, V, gate=True)
    x, gw = _rnd(dev, batch, heads * V), _rnd(dev, 2 * heads, heads * V) * 0.02
    n, mx, w = torch.zeros(batch, heads, K, device=dev), torch.zeros(batch, heads, device=dev), _rnd(dev, heads * V)
    ms = _median_ms(lambda: L.mlstm_step(q, k, v, x, gw, b, b, 15.0, m["slots"], m["starts"], m["S"], n, mx, heads, K, V, g, w, 1e-6), iters)
    return _line(ms, pk, nbytes=m["S"].numel() * 8 + n.numel() * 8 + batch * heads * (2 * K + 3 * V) * 2)


def kernel_conv(dev, pk, iters=20, seqs=16, tokens=16384, width=4096, taps=4):
    from minivllm_b200.layers.short_conv import conv_add
    m, cu = _state(dev, seqs, 1, 1, 1), _cu(_lens(seqs, tokens), dev)
    u, w, kept = _rnd(dev, tokens, width), _rnd(dev, width, taps), _rnd(dev, seqs, taps - 1, width)
    ms = _median_ms(lambda: conv_add(u, w, None, cu, m["slots"], m["starts"], kept), iters)
    return _line(ms, pk, nbytes=tokens * width * 4)


def kernel_stream_step(dev, pk, iters=20, rows=16384, width=2048, streams=2, taps=0):
    """taps > 0: rows are single tokens, with their convolution."""
    from minivllm_b200.layers import streams as ST
    from minivllm_b200.utils.context import reset_context, set_context
    x, y = torch.zeros(rows, streams, width, device=dev), _rnd(dev, rows, width)
    w, mix, out = _rnd(dev, width), _rnd(dev, streams, streams) * 0.3, _rnd(dev, streams)
    conv = None
    if taps:
        conv = ST.InputConvolution(_rnd(dev, width, taps))
        conv.slot_state = {"h": _rnd(dev, rows, taps - 1, width)}
        set_context(False, num_decode=rows, state_slots=torch.arange(rows, dtype=torch.int32, device=dev),
                    state_starts=torch.ones(rows, dtype=torch.int32, device=dev))
    entry = ST.StreamEntry(out, w, w, 1e-6, conv)
    ms = _median_ms(lambda: ST.stream_step(x, y, mix, out, entry), iters)
    reset_context()
    return _line(ms, pk, nbytes=rows * width * (8 * streams + 4 + (4 * (taps - 1) if taps else 0)))


def kernel_head_norm(dev, pk, iters=20, rows=16384, heads=16, vdim=128):
    from minivllm_b200.layers import group_norm as GN
    y, z, w, den = _rnd(dev, rows, heads * vdim), _rnd(dev, rows, heads * vdim), _rnd(dev, heads * vdim), torch.ones(rows, heads, device=dev)
    ms = _median_ms(lambda: GN.head_norm_gate(y, z, w, heads, 1e-6, den=den, act="sigmoid"), iters)
    return _line(ms, pk, nbytes=rows * heads * (vdim * 6 + 4))


# kernel -> (what runs it, the like kernel of Fozerax in bench_fozerax.KERNELS)
KERNELS = {
    "window_prefill_32seq_16heads": (kernel_window_prefill, "window_prefill_32seq_16heads"),
    "window_decode_b64_16heads": (kernel_window_decode, "window_decode_b64_16heads"),
    "qkv_rope_store_16384tok": (kernel_rope_store, "kv_norm_store_16384tok"),
    "mlstm_scan_16x1024tok": (kernel_mlstm_scan, "gla_scan_16x1024tok"),
    "mlstm_scan_1x16384tok": (lambda d, p, iters=20: kernel_mlstm_scan(d, p, iters, seqs=1), "gla_scan_1x16384tok"),
    "mlstm_gates_16x1024tok": (kernel_mlstm_gates, None),
    "mlstm_gates_1x16384tok": (lambda d, p, iters=20: kernel_mlstm_gates(d, p, iters, seqs=1), None),
    "mlstm_step_b64": (kernel_mlstm_step, "gla_step_b64"),
    "conv_add_16384tok": (kernel_conv, "conv_silu_16384tok"),
    "stream_step_16384x2x2048": (kernel_stream_step, "post_residual_norm_16384x2048"),
    "stream_step_16384x4x2048": (lambda d, p, iters=20: kernel_stream_step(d, p, iters, streams=4), "post_residual_norm_16384x2048"),
    "stream_step_and_conv_4096x2x2048": (lambda d, p, iters=20: kernel_stream_step(d, p, iters, rows=4096, taps=4), "post_residual_norm_16384x2048"),
    "head_norm_gate_16384x2048": (kernel_head_norm, "head_norm_gate_16384x2048"),
    "relu_glu_16384x4096": (lambda d, p, iters=20: BF.kernel_glu(d, p, iters, act="relu"), "gelu_glu_16384x4096"),
}


def run(device, pk, steps, only=None):
    from minivllm_b200.layers.attention import prefill_error_code
    kernels, like = {}, {}
    frac = lambda d: max(d.get("frac_hbm", 0.0), d.get("frac_bf16", 0.0))
    for name, (fn, other) in KERNELS.items():
        if only and only != name:
            continue
        kernels[name] = fn(device, pk, iters=max(5, steps))
        if other and other not in like:
            like[other] = BF.KERNELS[other][0](device, pk, iters=max(5, steps))
        torch.cuda.empty_cache()
        if other:
            kernels[name].update(like=other, like_us=like[other]["us"], like_frac=frac(like[other]),
                                 frac_over_like=frac(kernels[name]) / frac(like[other]))
    sizes = {}
    if not only:
        for name in SIZES:
            sizes[name] = {"dafotar": family_throughput(dafotar_config(name)), "fozerax": family_throughput(fozerax_config(name))}
    head = sizes.get("w2048", {}).get("dafotar", {})
    return {"metric": "Dafotar prefill tokens/s, width 2048, 4 layers, one wave of 16 x 1024 tokens",
            "value": head.get("prefill_tok_s"), "unit": "tok/s", "n_gpus": 1, "steps": steps, "warmup": 3,
            "higher_is_better": True, "data": "synthetic", "dtype": "bf16",
            "config": {"workload": "dafotar family beside the fozerax family at equal size; kernels at the shapes of width 2048"},
            "extra": {"throughput": sizes, "kernels": kernels, "error_word": prefill_error_code(device)}}
