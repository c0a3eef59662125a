"""Every mechanism of the Fozerax family alone, on the GPU, against the plain oracle's function for it."""
import pytest
import torch

from oracle import fozerax_oracle as oracle

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
IDS = ["fp32", "bf16"]
TOL = {torch.float32: 2e-6, torch.bfloat16: 8e-3}


def _rnd(seed, *shape, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def _close(got, want, tol, what=""):
    """Largest difference, relative to the largest entry."""
    got, want = got.double().cpu(), want.double()
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))
    assert err < tol, f"{what}: {err:.2e} (limit {tol:.1e})"


def _cu(lens):
    return torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32, device="cuda")


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------------------------------------ norms and gates
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width", [90, 64, 2048, 1536, 4096, 8192, 41])
def test_residual_steps(width, dtype):
    """A norm on the result only, the pair of mixers, and the normed embedding, with and without a norm behind them."""
    from minivllm_b200.layers import group_norm as GN
    rows, eps = 5, 1e-4
    a, b = _rnd(1, rows, width, dtype=dtype), _rnd(2, rows, 2 * width, dtype=dtype, scale=3.0)[:, width:]
    wa, wb, w1, w2 = (_rnd(i, width, dtype=dtype) for i in (3, 4, 5, 6))
    x, d = _rnd(7, rows, width), lambda t: t.double()
    norm = lambda t, w: oracle.rms_norm(d(t), d(w), eps)
    tol_x = 2e-6 if dtype == torch.float32 else 2e-5
    for w_next in (None, w2):
        nxt = w_next.cuda() if w_next is not None else None
        after = lambda t: oracle.rms_norm(t, d(w_next), eps) if w_next is not None else t
        want = d(x) + norm(a, w1)
        gx = x.cuda()
        h = GN.gated_residual_norm(gx, a.cuda(), None, None, w1.cuda(), nxt, 1.0, 1, eps)
        _close(gx, want, tol_x, "single")
        _close(h, after(want), TOL[dtype], "single, next")
        want = d(x) + norm(0.5 * (norm(a, wa) + norm(b, wb)), w1)
        gx = x.cuda()
        h = GN.pair_residual_norm(gx, a.cuda(), wa.cuda(), b.cuda(), wb.cuda(), w1.cuda(), nxt, 1.0, 1, eps)
        _close(gx, want, tol_x, "pair")
        _close(h, after(want), TOL[dtype], "pair, next")
        table, ids = _rnd(8, 11, width, dtype=dtype), torch.tensor([3, 0, 10, 3, 7])
        gx, h = GN.embed_norm(ids.cuda(), table.cuda(), nxt, 1, eps, w_post=w1.cuda())
        _close(gx, norm(table[ids], w1), tol_x, "embedding")
        _close(h, after(norm(table[ids], w1)), TOL[dtype], "embedding, next")
        pos = torch.randperm(rows * 2, generator=torch.Generator().manual_seed(8)).to(torch.int32).view(rows, 2)
        er, tw, sh = _rnd(9, rows * 2, width, dtype=dtype), _rnd(10, rows, 2).abs(), _rnd(11, rows, width, dtype=dtype)
        want = d(x) + norm((d(tw)[..., None] * d(er)[pos.long()]).sum(1) + d(sh), w1)
        gx = x.cuda()
        h = GN.moe_residual_norm(gx, er.cuda(), pos.cuda(), tw.cuda(), sh.cuda(), None, None, None, w1.cuda(), nxt, 1.0, 1, eps)
        _close(gx, want, tol_x, "experts")
        _close(h, after(want), TOL[dtype], "experts, next")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,vdim", [(3, 10), (4, 64), (1, 40), (12, 8), (16, 128), (2, 256)])
def test_head_norm_and_gate(heads, vdim, dtype):
    from minivllm_b200.layers import group_norm as GN
    n, eps = 6, 1e-3
    y, z, w = _rnd(1, n, heads * vdim, dtype=dtype), _rnd(2, n, heads * vdim + 8, dtype=dtype)[:, 8:], _rnd(3, vdim, dtype=dtype)
    want = oracle.rms_norm(y.double().view(n, heads, vdim), w.double(), eps).reshape(n, -1) * oracle.silu(z.double())
    _close(GN.head_norm_gate(y.cuda(), z.cuda(), w.cuda(), heads, eps), want, TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_activations(dtype):
    """The tanh form of gelu and the clamped gate, on both sides of every clamp."""
    from minivllm_b200.layers import group_norm as GN
    g, u = _rnd(1, 9, 77, dtype=dtype, scale=4.0), _rnd(2, 9, 77, dtype=dtype, scale=4.0)
    d = lambda t: t.double()
    _close(GN.gate_mul(u.cuda(), g.cuda(), "gelu_tanh"), oracle.gelu_tanh(d(g)) * d(u), TOL[dtype])
    for limit in (0.5, 3.0):
        got = GN.gate_mul(u.cuda(), g.cuda(), "clamped", limit=limit)
        _close(got, oracle.clamped_glu(d(g), d(u), limit), TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("experts,top,width,ff,tokens", [(5, 2, 72, 40, 33), (8, 3, 64, 128, 200), (3, 1, 90, 21, 10), (4, 4, 136, 72, 3)])
def test_experts_with_a_clamp(experts, top, width, ff, tokens, dtype):
    from minivllm_b200.layers import moe
    h, limit = _rnd(1, tokens, width, dtype=dtype), 0.8
    gate, up = _rnd(2, experts, ff, width, dtype=dtype, scale=1.5 * width ** -0.5), _rnd(3, experts, ff, width, dtype=dtype, scale=1.5 * width ** -0.5)
    idx, _ = moe.route(_rnd(4, tokens, experts).cuda(), None, top)
    pos, rows, offsets = moe.sort_by_expert(idx, experts)
    x = moe.gather_rows(h.cuda(), rows)
    w = torch.cat([gate, up], 1).cuda()
    forms = [False] + ([True] if dtype == torch.bfloat16 and width % 8 == 0 else [])
    for tc in forms:
        got = moe.grouped_linear(x, w, offsets, gated=True, tensor_cores=tc, act="clamped", limit=limit).cpu()
        for t in range(tokens):
            for k in range(top):
                e = int(idx[t, k])
                want = oracle.clamped_glu(gate[e].double() @ h[t].double(), up[e].double() @ h[t].double(), limit)
                _close(got[int(pos[t, k])], want, 1e-5 if dtype == torch.float32 else 1.6e-2, f"token {t}")


@pytest.mark.parametrize("experts,top,count,keep", [(10, 3, 5, 3), (9, 2, 3, 2), (8, 1, 8, 1), (8, 4, 2, 1), (6, 3, 1, 1), (6, 3, 3, 3),
                                                    (64, 6, 8, 3), (96, 5, 48, 7), (300, 8, 10, 4)])
def test_routing_in_groups(experts, top, count, keep):
    from minivllm_b200.layers import moe
    z = _rnd(experts + top, 57, experts, scale=2.0)
    # the best expert of all but one token's groups is far ahead; in token 0 the runner-up overall sits in a dropped group
    z[0] = -5.0
    size = experts // count
    for gnum in range(count):
        z[0, gnum * size] = 10.0 - gnum
        if size > 1:
            z[0, gnum * size + 1] = -20.0 + gnum
    idx, weight = moe.route(z.cuda(), None, top, count, keep)
    want_idx, want = oracle.route(z.double(), top, {"count": count, "keep": keep})
    assert torch.equal(idx.cpu().long(), want_idx)
    _close(weight, want, 1e-6)
    with pytest.raises(ValueError):
        moe.route(z.cuda(), None, experts // count * keep + 1, count, keep)


# ------------------------------------------------------------------------------------------------ windowed attention
def test_distance_bias_table():
    from minivllm_b200.layers import window_attention as WA
    for buckets, bias_max, window in ((10, 23, 11), (32, 110, 1 << 30), (16, 64, 40), (7, 12, 100), (8, 5, 64), (32, 200, 17)):
        rel = _rnd(buckets, buckets, 3)
        got = WA.distance_bias(rel, bias_max, window)
        far = min(window, 3 * bias_max)
        for n in range(far):
            want = rel[oracle.distance_bucket(n, buckets, bias_max)]
            assert torch.equal(got[:, min(n, got.shape[1] - 1)], want), (buckets, bias_max, n)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("qn,kn,vn", [(30, 14, 22), (64, 32, 16), (2048, 512, 512), (4096, 1024, 640), (1, 1, 1), (8, 8, 8)])
def test_norm_and_store(qn, kn, vn, dtype):
    from minivllm_b200.layers import window_attention as WA
    n, eps, pad = 5, 1e-3, -(qn + kn + vn) % 8
    p = _rnd(1, n, qn + kn + vn + pad, dtype=dtype)
    wq, wk = _rnd(2, qn, dtype=dtype), _rnd(3, kn, dtype=dtype)
    q, k, v = p[:, :qn].clone(), p[:, qn:qn + kn].clone(), p[:, qn + kn:qn + kn + vn].clone()
    cache, slots = torch.full((4, 8, kn + vn), 7.0, dtype=dtype, device="cuda"), torch.tensor([9, -1, 0, 31, 12])
    g = p.cuda()
    packed = WA.kv_norm_store(g[:, :qn], g[:, qn:qn + kn], g[:, qn + kn:qn + kn + vn], wq.cuda(), wk.cuda(), eps, cache,
                              slots.cuda(), packed=True)
    _close(g[:, :qn], oracle.rms_norm(q.double(), wq.double(), eps), TOL[dtype], "queries")
    _close(packed[:, :kn], oracle.rms_norm(k.double(), wk.double(), eps), TOL[dtype], "keys")
    assert torch.equal(packed[:, kn:].cpu(), v) and torch.equal(g[:, qn:].cpu(), p[:, qn:])
    flat = cache.view(32, -1)
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(flat[s], packed[i])
    assert bool((flat[[s for s in range(32) if s not in slots.tolist()]] == 7.0).all())


def _paged(rows, bs, dtype, seed=0, spare=3):
    """Rows of several sequences in a paged cache with shuffled blocks; rows that nobody owns are large."""
    g = torch.Generator().manual_seed(seed)
    need = [-(-r.shape[0] // bs) for r in rows]
    perm = torch.randperm(sum(need) + spare, generator=g).tolist()
    cache = torch.full((sum(need) + spare, bs, rows[0].shape[1]), 50.0, dtype=dtype)
    tables = torch.full((len(need), max(need)), -1, dtype=torch.int32)
    for s, r in enumerate(rows):
        for b in range(need[s]):
            phys = perm.pop()
            tables[s, b] = phys
            part = r[b * bs:(b + 1) * bs]
            cache[phys, :part.shape[0]] = part
    return cache.cuda(), tables.cuda()


def _sequences(lens, H, G, d, vd, dtype, seed, marked):
    """q, k, v per sequence.  All queries share a direction; keys are small except those at `marked` places, which point
    along it and carry a value of their own, so that whether a marked key is seen decides the output."""
    out = []
    e = _rnd(99, d)
    e = e / e.norm() * d ** 0.5
    for s, n in enumerate(lens):
        q = e + 0.1 * _rnd(seed + s, n, H, d)
        k, v = 0.3 * _rnd(seed + 50 + s, n, G, d), _rnd(seed + 100 + s, n, G, vd)
        for j in marked:
            if j < n:
                k[j] = e
                v[j] = 8.0 * _rnd(seed + 7 * j, G, vd)
        out.append((q.to(dtype), k.to(dtype), v.to(dtype)))
    return out


def _bias_of(rel, bias_max, window):
    from minivllm_b200.layers import window_attention as WA
    return WA.distance_bias(rel, bias_max, window).cuda()


WINDOW_CASES = [   # heads, kv heads, dim, vdim, window, bias_max, buckets, block
    (6, 2, 18, 13, 11, 23, 10, 16), (4, 1, 64, 128, 33, 40, 16, 64), (8, 4, 128, 64, 130, 300, 32, 16),
    (2, 2, 96, 64, 1, 20, 8, 8), (20, 1, 40, 24, 128, 60, 12, 32), (3, 3, 192, 128, 64, 64, 32, 16),
    (2, 1, 200, 160, 100, 90, 20, 64), (4, 2, 64, 64, 5000, 77, 32, 16), (4, 2, 136, 72, 257, 2000, 32, 48)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("case", WINDOW_CASES, ids=lambda c: "x".join(map(str, c)))
def test_window_attention(case, dtype):
    """Every kernel form on every token: prompts at once, portions behind cached tokens, single tokens; marked keys at
    block and tile borders, seen up to exactly one window later."""
    from minivllm_b200 import _cabi
    from minivllm_b200.layers import window_attention as WA
    from minivllm_b200.layers.latent_attention import latent_gather
    H, G, d, vd, window, bias_max, buckets, bs = case
    lens, scale, tol = [300, 1, 130, 77], 0.8 * d ** -0.5, 1e-5 if dtype == torch.float32 else 1.6e-2
    marked = [0, bs - 1, bs, 63, 64, 127, 128, 200]
    seqs = _sequences(lens, H, G, d, vd, dtype, 3, marked)
    rel, sink = _rnd(5, buckets, H).to(dtype), _rnd(6, H, scale=2.0).to(dtype)
    bias = _bias_of(rel, bias_max, window)
    want = [oracle.windowed_attention(q.double(), k.double(), v.double(), rel.double(), sink.double(), scale, window, bias_max)
            for q, k, v in seqs]
    rows = [torch.cat([k.reshape(len(k), -1), v.reshape(len(v), -1)], 1) for _, k, v in seqs]
    cache, tables = _paged(rows, bs, dtype)
    args = (G, d, vd, window, scale, bias, sink.cuda())
    tiles = dtype == torch.bfloat16 and bias.shape[1] <= _cabi.lib().mv_window_prefill_distances(d, vd)
    assert tiles or dtype == torch.float32 or d % 8 or vd % 8 or d > 192 or vd > 128
    flat_q = torch.cat([q.reshape(len(q), -1) for q, _, _ in seqs]).cuda()
    flat_want = torch.cat([w.reshape(len(w), -1) for w in want])
    pos = torch.cat([torch.arange(n) for n in lens]).cuda()
    cu = _cu(lens)
    _close(WA.window_attention_rows(flat_q, cache, tables, cu, pos, *args), flat_want, tol, "rows")
    if tiles:
        _close(WA.window_prefill(flat_q, torch.cat(rows).cuda(), cu, cu, *args), flat_want, tol, "prefill, whole")
    # portions: the last n tokens of every sequence behind what is cached
    for part in (2, 31, 76):
        take = [min(part, n) for n in lens]
        sel = torch.cat([torch.arange(n - t, n) + sum(lens[:s]) for s, (n, t) in enumerate(zip(lens, take))])
        cu_q = _cu(take)
        got = WA.window_attention_rows(flat_q[sel.cuda()], cache, tables, cu_q, pos[sel.cuda()], *args)
        _close(got, flat_want[sel], tol, f"rows, portion of {part}")
        if tiles:
            first = [max(0, n - t - window + 1) for n, t in zip(lens, take)]
            keys = [n - f for n, f in zip(lens, first)]
            packed = latent_gather(cache, _cu(keys), sum(keys), tables, _i32(first))
            assert torch.equal(packed.cpu(), torch.cat([r[f:] for r, f in zip(rows, first)]))
            got = WA.window_prefill(flat_q[sel.cuda()], packed, cu_q, _cu(keys), *args)
            _close(got, flat_want[sel], tol, f"prefill, portion of {part}")
    # decoded tokens: every place of the longest sequence in turn as one batch, and few sequences (the window in pieces)
    places = sorted({p for m in marked for p in (m, m + 1, m + window - 1, m + window) if p < lens[0]} | {299})
    for batch in (places, places[-2:]):
        q = flat_q[torch.tensor(batch).cuda()]
        at = torch.tensor(batch).cuda()
        tab = tables[:1].expand(len(batch), -1).contiguous()
        ref = flat_want[batch]
        _close(WA.window_attention_rows(q, cache, tab, None, at, *args), ref, tol, "rows, one token each")
        got = WA.window_decode(q, cache, tab, at, *args)
        assert (got is None) == (dtype == torch.float32 or bool(d % 8 or vd % 8))
        if got is not None:
            _close(got, ref, tol, "decode")
    assert int(WA._error_word(flat_q.device).item()) == 0


def test_window_attention_without_bias_or_sink_and_padding_rows():
    from minivllm_b200.layers import window_attention as WA
    H, G, d, vd, bs, window = 4, 2, 64, 64, 16, 20
    (q, k, v), = _sequences([150], H, G, d, vd, torch.bfloat16, 9, [40])
    rows = torch.cat([k.reshape(150, -1), v.reshape(150, -1)], 1)
    cache, tables = _paged([rows], bs, torch.bfloat16)
    want = oracle.windowed_attention(q.double(), k.double(), v.double(), torch.zeros(4, H, dtype=torch.float64),
                                     torch.full((H,), -1e9, dtype=torch.float64), 0.125, window, 50).reshape(150, -1)
    qf, cu = q.reshape(150, -1).cuda(), _cu([150])
    args = (G, d, vd, window, 0.125)
    _close(WA.window_prefill(qf, rows.cuda(), cu, cu, *args), want, 1.6e-2, "prefill")
    pos = torch.tensor([149, -1, 41, 59, 60]).cuda()
    tab = tables.expand(5, -1).clone()
    tab[1] = -1
    got = WA.window_decode(qf[pos.clamp_min(0)], cache, tab, pos, *args)
    assert bool((got[1] == 0).all())
    _close(got[[0, 2, 3, 4]], want[[149, 41, 59, 60]], 1.6e-2, "decode")


# ------------------------------------------------------------------------------------------------ recurrences
def _run_portions(fn, lens, cuts):
    """Calls fn(spans) with spans = [(sequence, from, to)] until every sequence is through, cutting as `cuts` says."""
    at, k = [0] * len(lens), 0
    while any(a < n for a, n in zip(at, lens)):
        spans = []
        for s, n in enumerate(lens):
            step = min(cuts[(k + s) % len(cuts)], n - at[s])
            if step:
                spans.append((s, at[s], at[s] + step))
                at[s] += step
        fn(spans)
        k += 1


SCAN_SIZES = [(2, 14, 10), (1, 37, 41), (3, 64, 64), (2, 128, 128), (1, 96, 36), (2, 32, 200), (1, 130, 20), (1, 256, 64), (4, 8, 8), (1, 1, 3),
              (2, 48, 132), (1, 200, 300), (2, 96, 40), (1, 128, 256), (2, 16, 136)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,K,V", SCAN_SIZES)
def test_gla_scan(heads, K, V, dtype):
    """Portions and single tokens from slots whose old contents must not be seen; channels that forget at once beside
    channels that never do."""
    from minivllm_b200.layers import gla as L
    lens, tau, eps = [70, 1, 33], 3.0, 1e-4
    seqs = []
    for s, n in enumerate(lens):
        q, k, v, g = (_rnd(10 * s + i, n, heads, D, dtype=dtype) for i, D in enumerate((K, K, V, V)))
        z = _rnd(10 * s + 5, n, heads, K, scale=4.0) + 3.0
        z[:, :, 0] = -60.0
        z[:, :, -1] = 30.0
        seqs.append((q, k, v, g, z.to(dtype)))
    w = _rnd(77, V, dtype=dtype)
    d = lambda t: t.double()
    ref = [oracle.gla_scan(d(q) * K ** -0.5, d(k), d(v), oracle.channel_decay(d(z), tau)) for q, k, v, g, z in seqs]
    gated = [(oracle.rms_norm(o, d(w), eps) * oracle.silu(d(x[3]))).flatten(1) for (o, _), x in zip(ref, seqs)]
    slots, tol = [4, 0, 2], 3e-6 if dtype == torch.float32 else 6e-3
    for cuts in ([100], [7, 1, 2, 16], [1]):
        state = torch.full((6, heads, K, V), float("nan"), device="cuda")

        def step(spans):
            cat = lambda i: torch.cat([seqs[s][i][a:b].flatten(1) for s, a, b in spans])
            p = torch.cat([cat(0), cat(1), cat(2), cat(3)], 1).cuda()
            q, k, v, g = p.split([heads * K, heads * K, heads * V, heads * V], 1)
            z, sl, st = cat(4).cuda(), _i32([slots[s] for s, _, _ in spans]), _i32([a for _, a, _ in spans])
            single = all(b - a == 1 for _, a, b in spans)
            cu = None if single else _cu([b - a for _, a, b in spans])
            got = L.gla_scan(q, k, v, z, tau, cu, sl, st, state, heads, K, V, gate=g, norm_w=w.cuda(), eps=eps)
            want = torch.cat([(gated[s] if single else ref[s][0].flatten(1))[a:b] for s, a, b in spans])
            _close(got, want, tol * (3 if single else 1), f"cuts {cuts}, {spans}")

        _run_portions(step, lens, cuts)
        for s in range(len(lens)):
            _close(state[slots[s]], ref[s][1], 3e-6 if dtype == torch.float32 else 1e-4, "state")
        assert bool(state[[1, 3, 5]].isnan().all())


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,K,V", SCAN_SIZES)
def test_delta_scan(heads, K, V, dtype):
    """The same for the delta rule, with its convolution; one head forgets almost everything, one nothing."""
    from minivllm_b200.layers import gated_delta as L
    from minivllm_b200.layers.short_conv import conv_silu, conv_state_update
    taps, eps, lens = 1 + heads, 1e-4, [70, 1, 33]
    kv = heads if heads % 2 else heads // 2
    ch = 2 * kv * K + heads * V
    conv_w, A_log, dt_bias, w = _rnd(1, ch, taps, dtype=dtype), _rnd(2, heads, dtype=dtype), _rnd(3, heads, dtype=dtype), _rnd(4, V, dtype=dtype)
    A_log[0], A_log[-1] = (4.0, A_log[-1]) if heads > 1 else (A_log[0], A_log[0])
    if heads > 1:
        A_log[-1] = -12.0
    seqs = [(_rnd(20 + s, n, ch, dtype=dtype), _rnd(30 + s, n, heads, dtype=dtype), _rnd(40 + s, n, heads, dtype=dtype),
             _rnd(50 + s, n, heads * V, dtype=dtype)) for s, n in enumerate(lens)]
    d = lambda t: t.double()
    rnd = lambda t: t.to(dtype).double()          # the convolution's result is kept in the model's type
    ref, gated = [], []
    for u, b, a, g in seqs:
        x = rnd(oracle.causal_conv_silu(d(u), d(conv_w)))
        spread = lambda t: t.reshape(len(u), kv, K).repeat_interleave(heads // kv, 1)
        o, S = oracle.delta_scan(oracle.unit(spread(x[:, :kv * K])) * K ** -0.5, oracle.unit(spread(x[:, kv * K:2 * kv * K])),
                                 x[:, 2 * kv * K:].reshape(len(u), heads, V), oracle.sigmoid(d(b)),
                                 oracle.head_decay(d(a), d(A_log), d(dt_bias)))
        ref.append((o.flatten(1), S))
        gated.append((oracle.rms_norm(o, d(w), eps)).flatten(1) * oracle.silu(d(g)))
    slots, tol = [4, 0, 2], 5e-6 if dtype == torch.float32 else 1.2e-2
    for cuts in ([100], [7, 1, 2, 16], [1]):
        state = torch.full((6, heads, K, V), float("nan"), device="cuda")
        conv = torch.full((6, taps - 1, ch), float("nan"), dtype=dtype, device="cuda")

        def step(spans):
            cat = lambda i: torch.cat([seqs[s][i][lo:hi] for s, lo, hi in spans]).cuda()
            u, ba, g = cat(0), torch.cat([cat(1), cat(2)], 1), cat(3)
            sl, st = _i32([slots[s] for s, _, _ in spans]), _i32([lo for _, lo, _ in spans])
            single = all(hi - lo == 1 for _, lo, hi in spans)
            cu = _cu([hi - lo for _, lo, hi in spans])
            x = u if single else conv_silu(u, conv_w.cuda(), None, cu, sl, st, conv)
            got = L.delta_scan(x, ba[:, :heads], ba[:, heads:], A_log.cuda(), dt_bias.cuda(), None if single else cu, sl, st,
                               state, heads, kv, K, V, conv_w=conv_w.cuda(), conv_state=conv, gate=g, norm_w=w.cuda(), eps=eps)
            conv_state_update(conv, u, taps, cu, sl, st)
            want = torch.cat([(gated[s] if single else ref[s][0])[lo:hi] for s, lo, hi in spans])
            _close(got, want, tol * (4 if single else 1), f"cuts {cuts}, {spans}")

        _run_portions(step, lens, cuts)
        for s in range(len(lens)):
            _close(state[slots[s]], ref[s][1], 5e-6 if dtype == torch.float32 else 1.2e-2, "state")
        assert bool(state[[1, 3, 5]].isnan().all())


@pytest.mark.parametrize("K,V", [(64, 64), (128, 128), (32, 24), (96, 72), (128, 256), (8, 200)])
def test_chunked_scans(K, V):
    """The chunked kernels against the oracle: lengths around the chunk size, cuts inside chunks, one sequence and several,
    channels that forget at once; nothing of the state is rounded to 16 bits."""
    from minivllm_b200.layers import gated_delta as D
    from minivllm_b200.layers import gla as L
    bf, d = torch.bfloat16, lambda t: t.double()
    H, kv, tau = 2, 1, 2.0
    for lens in ([1, 63, 64, 65, 130, 2], [200]):
        z = [(_rnd(5 + s, n, H, K, scale=3.0) + 3.0).to(bf) for s, n in enumerate(lens)]
        for x in z:
            x[:, :, 0] = -70.0                   # alpha of 2^-50
            x[:, :, 1::5] = 12.0                 # alpha close to one
        g = [torch.cat([_rnd(20 + s, n, 2 * H * K), _rnd(40 + s, n, H * V)], 1).to(bf) for s, n in enumerate(lens)]
        u = [torch.cat([_rnd(60 + s, n, 2 * kv * K), _rnd(80 + s, n, H * V)], 1).to(bf) for s, n in enumerate(lens)]
        ba = [torch.cat([_rnd(100 + s, n, H, scale=2.0), _rnd(120 + s, n, H)], 1).to(bf) for s, n in enumerate(lens)]
        A_log, dt_bias = torch.tensor([-3.0, 3.0]).to(bf), torch.tensor([-1.0, 0.5]).to(bf)
        ref_g, ref_d = [], []
        for s, n in enumerate(lens):
            q, k, v = d(g[s]).split([H * K, H * K, H * V], 1)
            ref_g.append(oracle.gla_scan(q.view(n, H, K) * K ** -0.5, k.view(n, H, K), v.view(n, H, V), oracle.channel_decay(d(z[s]), tau)))
            q, k, v = d(u[s]).split([kv * K, kv * K, H * V], 1)
            spread = lambda t: t.view(n, kv, K).repeat_interleave(H // kv, 1)
            ref_d.append(oracle.delta_scan(oracle.unit(spread(q)) * K ** -0.5, oracle.unit(spread(k)), v.view(n, H, V),
                                           oracle.sigmoid(d(ba[s][:, :H])), oracle.head_decay(d(ba[s][:, H:]), d(A_log), d(dt_bias))))
        for cuts in ([400], [70, 3, 64, 1], [37]):
            Sg, Sd = (torch.full((len(lens), H, K, V), float("nan"), device="cuda") for _ in range(2))

            def step(spans):
                cat = lambda x: torch.cat([x[s][a:b] for s, a, b in spans]).cuda()
                sl, st, cu = _i32([s for s, _, _ in spans]), _i32([a for _, a, _ in spans]), _cu([b - a for _, a, b in spans])
                q, k, v = cat(g).split([H * K, H * K, H * V], 1)
                got = L.gla_scan(q, k, v, cat([x.flatten(1) for x in z]), tau, cu, sl, st, Sg, H, K, V, chunked=True)
                _close(got, torch.cat([ref_g[s][0][a:b].flatten(1) for s, a, b in spans]), 6e-3, f"gla, {lens}, {spans}")
                b = cat(ba)
                got = D.delta_scan(cat(u), b[:, :H], b[:, H:], A_log.cuda(), dt_bias.cuda(), cu, sl, st, Sd, H, kv, K, V, chunked=True)
                _close(got, torch.cat([ref_d[s][0][a:b].flatten(1) for s, a, b in spans]), 6e-3, f"delta, {lens}, {spans}")

            _run_portions(step, lens, cuts)
            for s in range(len(lens)):
                _close(Sg[s], ref_g[s][1], 1e-4, "gla, state")
                _close(Sd[s], ref_d[s][1], 1e-4, "delta, state")


def test_padding_rows_leave_the_state_alone():
    from minivllm_b200.layers import gated_delta as D
    from minivllm_b200.layers import gla as L
    H, K, V = 2, 16, 8
    state = torch.full((3, H, K, V), 2.0, device="cuda")
    p, z = _rnd(1, 2, 2 * H * K + 2 * H * V).cuda(), _rnd(2, 2, H * K).cuda()
    q, k, v, g = p.split([H * K, H * K, H * V, H * V], 1)
    out = L.gla_scan(q, k, v, z, 2.0, None, _i32([2, 1]), _i32([-1, 5]), state, H, K, V, gate=g, norm_w=_rnd(3, V).cuda(), eps=1e-5)
    assert bool((out[0] == 0).all()) and bool((out[1] != 0).any())
    u, ba = _rnd(4, 2, 2 * H * K + H * V).cuda(), _rnd(5, 2, 2 * H).cuda()
    conv = torch.full((3, 1, u.shape[1]), 2.0, device="cuda")
    out = D.delta_scan(u, ba[:, :H], ba[:, H:], _rnd(6, H).cuda(), _rnd(7, H).cuda(), None, _i32([2, 1]), _i32([-1, 5]), state, H, H,
                       K, V, conv_w=_rnd(8, u.shape[1], 2).cuda(), conv_state=conv, gate=g, norm_w=_rnd(9, V).cuda(), eps=1e-5)
    assert bool((out[0] == 0).all()) and bool((out[1] != 0).any())
    assert bool((state[[0, 2]] == 2.0).all()) and bool((state[1] != 2.0).any()) and bool((conv == 2.0).all())


def test_slow_decay_over_many_tokens():
    """A write at the start is read out 3,000 tokens later, through many portions."""
    from minivllm_b200.layers import gated_delta as D
    from minivllm_b200.layers import gla as L
    H, K, V, n = 1, 32, 16, 3000
    q, k, v = _rnd(1, n, K), _rnd(2, n, K, scale=1e-3), _rnd(3, n, V, scale=1e-3)
    k[0], v[0] = _rnd(4, K), _rnd(5, V)
    z = torch.full((n, K), 9.0)
    ref, S = oracle.gla_scan(q.double()[:, None] * K ** -0.5, k.double()[:, None], v.double()[:, None],
                             oracle.channel_decay(z.double(), 4.0)[:, None])
    state = torch.zeros(1, H, K, V, device="cuda")
    p = torch.cat([q, k, v], 1).cuda()
    outs = [L.gla_scan(p[a:a + 500, :K], p[a:a + 500, K:2 * K], p[a:a + 500, 2 * K:], z[a:a + 500].cuda(), 4.0, _cu([500]), _i32([0]),
                       _i32([a]), state, H, K, V) for a in range(0, n, 500)]
    _close(torch.cat(outs)[-500:], ref[-500:, 0], 1e-5, "gla, late")
    _close(state[0], S, 1e-5, "gla, state")
    qkv = torch.cat([q, k, v], 1)
    ba = torch.zeros(n, 2)
    ba[1:, 0] = -20.0                    # only the first token writes
    A_log, dt_bias = torch.tensor([-4.0]), torch.tensor([-4.0])
    ref, S = oracle.delta_scan((oracle.unit(q.double()) * K ** -0.5)[:, None], oracle.unit(k.double())[:, None], v.double()[:, None],
                               oracle.sigmoid(ba[:, :1].double()), oracle.head_decay(ba[:, 1:].double(), A_log.double(), dt_bias.double()))
    state.zero_()
    x, g = qkv.cuda(), ba.cuda()
    outs = [D.delta_scan(x[a:a + 500], g[a:a + 500, :1], g[a:a + 500, 1:], A_log.cuda(), dt_bias.cuda(), _cu([500]), _i32([0]), _i32([a]),
                         state, H, 1, K, V) for a in range(0, n, 500)]
    _close(torch.cat(outs)[-500:], ref[-500:, 0], 1e-5, "delta, late")
    _close(state[0], S, 1e-5, "delta, state")
