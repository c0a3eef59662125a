"""`bench.py --workload sipazen`: throughput of the Sipazen family beside the Qwen3-shaped family at equal size, and
every kernel of the family against its roofline.

Sizes: random weights, four layers (two latent-attention, two state-space), experts of a mid-size mixture.  The
Qwen3-shaped model of a size has the same width, layer count and vocabulary, heads of 128 over the same width, and a
feed-forward as wide as the experts a token uses.  Prefill is one wave of 16 prompts x 1,024 tokens, decode the
captured graph with 64 sequences behind 1,024-token contexts; both timed on the device with CUDA events around the
engine's own step, per-step inputs of more than the L2 size (weights and cache).
"""
import torch


def _median_ms(fn, iters, warmup=3):
    """Median device time of single calls, queued behind a pause of some 20 ms so that the host's own time stays out of it."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    ev = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(iters)]
    torch.cuda._sleep(40_000_000)
    for a, b in ev:
        a.record()
        fn()
        b.record()
    torch.cuda.synchronize()
    ms = sorted(a.elapsed_time(b) for a, b in ev)
    return ms[len(ms) // 2]


SIZES = {
    "w1024": dict(width=1024, heads=8, rank=256, mheads=32, experts=32, top=4, ff=512, shared=1024),
    "w2048": dict(width=2048, heads=16, rank=512, mheads=64, experts=64, top=6, ff=1024, shared=2048),
    "w4096": dict(width=4096, heads=32, rank=512, mheads=128, experts=64, top=6, ff=1536, shared=3072),
}
VOCAB = 32768


def sipazen_config(s, **over):
    att = {"type": "latent_attention",
           "mixer": {"heads": s["heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": s["rank"],
                     "scale": 192 ** -0.5, "rot": {"base": 1e6, "dims": 64}}}
    ssm = {"type": "mamba2", "mixer": {"heads": s["mheads"], "vdim": 64, "state": 128, "groups": 8, "conv": 4,
                                       "norm_groups": 8}}
    mlp = {"kind": "moe", "router": {"experts": s["experts"], "top": s["top"]}, "expert": {"ff": s["ff"]},
           "shared": {"ff": s["shared"]}}
    c = {"architecture": "Sipazen", "vocab": VOCAB, "width": s["width"], "residual_mult": 0.5,
         "norm": {"eps": 1e-5, "groups": 4}, "layers": [{**l, "mlp": mlp} for l in (att, ssm, att, ssm)]}
    return {**c, **over}


def qwen_config(s, **over):
    heads = s["width"] // 128
    return {**dict(vocab_size=VOCAB, hidden_size=s["width"], num_layers=4, num_heads=heads, num_kv_heads=max(heads // 4, 1),
                   head_dim=128, intermediate_size=s["top"] * s["ff"] + s["shared"], tie_word_embeddings=False), **over}


def family_throughput(config, prompts=16, prompt_len=1024, batch=64, iters=10):
    from minivllm_b200.engine.llm_engine import LLMEngine
    from minivllm_b200.engine.sequence import Sequence
    eng = LLMEngine({**config, "max_model_length": 2048, "block_size": 256, "max_num_seqs": batch,
                     "num_kv_blocks": batch * 6, "max_num_batched_tokens": prompts * prompt_len, "greedy": True,
                     "dtype": torch.bfloat16})
    r, bm = eng.model_runner, eng.scheduler.block_manager
    g = torch.Generator().manual_seed(0)
    seqs = []
    for _ in range(batch):
        q = Sequence(torch.randint(0, VOCAB, (prompt_len,), generator=g).tolist(), block_size=256)
        bm.allocate(q)
        seqs.append(q)
    out = {}
    with torch.inference_mode():
        ms = _median_ms(lambda: r._prefill_body(seqs[:prompts], None), iters)
        out["prefill_ms"], out["prefill_tok_s"] = ms, prompts * prompt_len / ms * 1e3
        for i in range(0, batch, prompts):
            r._prefill_body(seqs[i:i + prompts], None)
        for q in seqs:
            for _ in range(8 * iters):
                q.append_token(0)
            bm.reserve(q)
        ms = _median_ms(lambda: r._replay(seqs, None), 4 * iters)
        out["decode_ms"], out["decode_tok_s"] = ms, batch / ms * 1e3
    eng.exit()
    del eng, r
    torch.cuda.empty_cache()
    return out


# ------------------------------------------------------------------------------------------------- kernels
def _line(ms, pk, nbytes=None, flops=None):
    d = {"us": ms * 1e3}
    if nbytes:
        d.update(GBps=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / pk["hbm_gbs"])
    if flops:
        d.update(TFLOPs=flops / ms / 1e9, frac_bf16=flops / ms / 1e9 / pk["bf16_tflops"])
    return d


def _cu(lens, dev):
    return torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)


def _tables(batch, ctx, bs, dev, seed=0):
    per = -(-max(ctx) // bs)
    perm = torch.randperm(batch * per, generator=torch.Generator().manual_seed(seed)).to(torch.int32)
    return perm.view(batch, per).to(dev), batch * per


def kernel_latent_prefill(dev, pk, iters=20, heads=16, dim=128, rot=64, vdim=128):
    from minivllm_b200.layers import latent_attention as LA
    from minivllm_b200 import synth
    lens = synth.prefill_inputs(num_seqs=32, len_lo=128, len_hi=2048)["lens"]
    lens = [int(n) for n in lens]
    T = sum(lens)
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev, dtype=torch.float32).to(torch.bfloat16)
    q, kv, kr, sink = rnd(T, heads * (dim + rot)), rnd(T, heads * (dim + vdim)), rnd(T, rot), rnd(heads)
    cu = _cu(lens, dev)
    ms = _median_ms(lambda: LA.latent_prefill(q, kv, kr, cu, cu, heads, dim, rot, vdim, 192 ** -0.5, sink), iters)
    pairs = sum(n * (n + 1) // 2 for n in lens)
    return _line(ms, pk, flops=2.0 * heads * (dim + rot + vdim) * pairs)


def kernel_latent_decode(dev, pk, iters=20, batch=64, heads=16, rank=512, rot=64):
    from minivllm_b200.layers import latent_attention as LA
    g = torch.Generator().manual_seed(0)
    ctx = torch.randint(1024, 4097, (batch,), generator=g).tolist()
    tables, blocks = _tables(batch, ctx, 64, dev)
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.float32).to(torch.bfloat16)
    cache = rnd(blocks, 64, rank + rot)
    ql, qr, sink = rnd(batch, heads, rank), rnd(batch, heads, rot), rnd(heads)
    pos = torch.tensor(ctx, device=dev, dtype=torch.int64) - 1
    ms = _median_ms(lambda: LA.latent_decode(ql, qr, cache, tables, pos, sink, 192 ** -0.5), iters)
    return _line(ms, pk, nbytes=sum(ctx) * (rank + rot) * 2 + batch * heads * (2 * rank + rot) * 2)


def kernel_grouped(dev, pk, tokens, gated, iters=20, experts=64, top=6, width=2048, ff=1024):
    from minivllm_b200.layers import moe
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.float32).to(torch.bfloat16)
    idx, _ = moe.route(torch.randn(tokens, experts, device=dev), None, top)
    _, _, offsets = moe.sort_by_expert(idx, experts)
    rows = tokens * top
    used = int((offsets[1:] > offsets[:-1]).sum())
    if gated:
        x, w = rnd(rows, width), rnd(experts, 2 * ff, width)
    else:
        x, w = rnd(rows, ff), rnd(experts, width, ff)
    ms = _median_ms(lambda: moe.grouped_linear(x, w, offsets, gated), iters)
    per = w.shape[1] * w.shape[2]
    out_dim = ff if gated else width
    return _line(ms, pk, nbytes=used * per * 2 + (x.numel() + rows * out_dim) * 2, flops=2.0 * rows * per)


def _mamba(dev, lens, heads=64, P=64, N=128, G=8):
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.float32).to(torch.bfloat16)
    T, ch = sum(lens), heads * P + 2 * G * N
    return dict(u=rnd(T, heads * P + ch + heads), dt=rnd(T, heads), cw=rnd(ch, 4), cb=rnd(ch), par=[rnd(heads) for _ in range(3)],
                slots=torch.arange(len(lens), dtype=torch.int32, device=dev),
                starts=torch.ones(len(lens), dtype=torch.int32, device=dev),
                conv=rnd(len(lens), 3, ch), ssm=torch.zeros(len(lens), heads, N, P, device=dev), cu=_cu(lens, dev),
                dims=(heads, P, N, G), ch=ch, inner=heads * P)


def kernel_conv(dev, pk, iters=20, tokens=16384):
    from minivllm_b200.layers import mamba2 as M
    m = _mamba(dev, [tokens // 16] * 16)
    u = m["u"][:, m["inner"]:m["inner"] + m["ch"]]
    ms = _median_ms(lambda: M.conv_silu(u, m["cw"], m["cb"], m["cu"], m["slots"], m["starts"], m["conv"]), iters)
    return _line(ms, pk, nbytes=tokens * m["ch"] * 4)


def kernel_chunk_scan(dev, pk, iters=20, seqs=16, tokens=16384):
    from minivllm_b200.layers import mamba2 as M
    m = _mamba(dev, [tokens // seqs] * seqs)
    xbc = torch.randn(tokens, m["ch"], device=dev).to(torch.bfloat16)
    H, P, N, G = m["dims"]
    ms = _median_ms(lambda: M.ssm_scan(xbc, m["dt"], *m["par"], m["cu"], m["slots"], m["starts"], m["ssm"], *m["dims"]), iters)
    q = 64      # products of the chunked form, every one once and in full
    flops = 2.0 * tokens * (H * (q * P + 2 * N * P) + G * q * N)
    return _line(ms, pk, nbytes=tokens * (2 * m["inner"] + 2 * G * N + H) * 2 + m["ssm"].numel() * 8, flops=flops)


def kernel_ssm_step(dev, pk, iters=20, batch=64):
    from minivllm_b200.layers import mamba2 as M
    m = _mamba(dev, [1] * batch)
    u = m["u"][:, m["inner"]:m["inner"] + m["ch"]]
    ms = _median_ms(lambda: M.ssm_step(u, m["cw"], m["cb"], m["conv"], m["dt"], *m["par"], m["slots"], m["starts"], m["ssm"],
                                       *m["dims"]), iters)
    return _line(ms, pk, nbytes=m["ssm"].numel() * 8)


def kernel_residual_norm(dev, pk, iters=20, rows=16384, width=2048):
    from minivllm_b200.layers import group_norm as GN
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.float32).to(torch.bfloat16)
    x, y, gate, b, w1, w2 = torch.zeros(rows, width, device=dev), rnd(rows, width), rnd(rows, width), rnd(width), rnd(width), rnd(width)
    ms = _median_ms(lambda: GN.gated_residual_norm(x, y, gate, b, w1, w2, 0.5, 4, 1e-5), iters)
    return _line(ms, pk, nbytes=rows * width * 14)


def kernel_moe_residual(dev, pk, iters=20, rows=16384, width=2048, top=6):
    from minivllm_b200.layers import group_norm as GN
    from minivllm_b200.layers import moe
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.float32).to(torch.bfloat16)
    x, y, gate, b, w1, w2 = torch.zeros(rows, width, device=dev), rnd(rows * top, width), rnd(rows, width), rnd(width), rnd(width), rnd(width)
    sh, sg = rnd(rows, width), rnd(rows, 8)
    idx, w = moe.route(torch.randn(rows, 64, device=dev), None, top)
    pos, _, _ = moe.sort_by_expert(idx, 64)
    ms = _median_ms(lambda: GN.moe_residual_norm(x, y, pos, w, sh, sg, gate, b, w1, w2, 0.5, 4, 1e-5), iters)
    return _line(ms, pk, nbytes=rows * width * (14 + 2 * top))


def kernel_gated_norm(dev, pk, iters=20, rows=16384, width=4096):
    from minivllm_b200.layers import group_norm as GN
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.float32).to(torch.bfloat16)
    y, z, w = rnd(rows, width), rnd(rows, width), rnd(width)
    ms = _median_ms(lambda: GN.gated_group_norm(y, z, w, 8, 1e-5), iters)
    return _line(ms, pk, nbytes=rows * width * 6)


def kernel_gate_mul(dev, pk, iters=20, rows=16384, cols=2048):
    from minivllm_b200.layers import group_norm as GN
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.float32).to(torch.bfloat16)
    y, g = rnd(rows, cols), rnd(rows, 2 * cols)[:, cols:]
    ms = _median_ms(lambda: GN.gate_mul(y, g), iters)
    return _line(ms, pk, nbytes=rows * cols * 6)


def kernel_latent_prep(dev, pk, iters=20, rows=16384, heads=16, dim=128, rot=64, rank=512):
    from minivllm_b200.layers import latent_attention as LA
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.float32).to(torch.bfloat16)
    q, down, w = rnd(rows, heads * (dim + rot)), rnd(rows, rank + rot), rnd(rank)
    cache = rnd(rows // 64, 64, rank + rot)
    pos, slots = torch.arange(rows, device=dev) % 1024, torch.arange(rows, device=dev)
    ct, st = LA.rope_table(1e6, rot, 2048, dev)
    ms = _median_ms(lambda: LA.latent_prep(q, down, w, pos, ct, st, heads, dim, rot, rot, rank, 1e-5, cache, slots), iters)
    return _line(ms, pk, nbytes=rows * (heads * rot * 2 + 3 * (rank + rot)) * 2)


def kernel_route_sort_gather(dev, pk, iters=20, tokens=16384, experts=64, top=6, width=2048):
    from minivllm_b200.layers import moe
    z, h = torch.randn(tokens, experts, device=dev), torch.randn(tokens, width, device=dev).to(torch.bfloat16)
    out = {"route": _line(_median_ms(lambda: moe.route(z, None, top), iters), pk, nbytes=tokens * (experts + 2 * top) * 4)}
    idx, _ = moe.route(z, None, top)
    out["sort"] = _line(_median_ms(lambda: moe.sort_by_expert(idx, experts), iters), pk, nbytes=tokens * top * 16)
    _, rt, _ = moe.sort_by_expert(idx, experts)
    out["gather"] = _line(_median_ms(lambda: moe.gather_rows(h, rt), iters), pk, nbytes=tokens * (top + 1) * width * 2)
    return out


KERNELS = {
    "latent_prefill_32seq_16heads": kernel_latent_prefill,
    "latent_decode_b64_16heads": kernel_latent_decode,
    "grouped_gate_up_16384tok": lambda d, p, iters=20: kernel_grouped(d, p, 16384, True, iters),
    "grouped_down_16384tok": lambda d, p, iters=20: kernel_grouped(d, p, 16384, False, iters),
    "grouped_gate_up_64tok": lambda d, p, iters=20: kernel_grouped(d, p, 64, True, iters),
    "grouped_down_64tok": lambda d, p, iters=20: kernel_grouped(d, p, 64, False, iters),
    "conv_silu_16384tok": kernel_conv,
    "ssm_chunk_scan_16x1024tok": kernel_chunk_scan,
    "ssm_chunk_scan_1x16384tok": lambda d, p, iters=20: kernel_chunk_scan(d, p, iters, seqs=1),
    "ssm_step_b64": kernel_ssm_step,
    "gated_residual_norm_16384x2048": kernel_residual_norm,
    "moe_residual_norm_16384x2048": kernel_moe_residual,
    "gated_group_norm_16384x4096": kernel_gated_norm,
    "gate_mul_16384x2048": kernel_gate_mul,
    "latent_prep_16384tok": kernel_latent_prep,
    "moe_route_sort_gather": kernel_route_sort_gather,
}


def run(device, pk, steps, only=None):
    from minivllm_b200.layers.attention import prefill_error_code
    kernels = {}
    for name, fn in KERNELS.items():
        if only and only != name:
            continue
        kernels[name] = fn(device, pk, iters=max(5, steps))
        torch.cuda.empty_cache()
    sizes = {}
    if not only:
        for name, s in SIZES.items():
            sizes[name] = {"sipazen": family_throughput(sipazen_config(s)), "qwen3": family_throughput(qwen_config(s))}
    head = sizes.get("w2048", {}).get("sipazen", {})
    return {"metric": "Sipazen prefill tokens/s, width 2048, 4 layers, one wave of 16 x 1024 tokens",
            "value": head.get("prefill_tok_s"), "unit": "tok/s", "n_gpus": 1, "steps": steps, "warmup": 3,
            "higher_is_better": True, "data": "synthetic", "dtype": "bf16",
            "config": {"workload": "sipazen family beside the qwen3 family at equal size; kernels at the shapes of width 2048"},
            "extra": {"throughput": sizes, "kernels": kernels, "error_word": prefill_error_code(device)}}
