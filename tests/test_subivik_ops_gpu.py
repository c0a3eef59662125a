"""Every mechanism of the Subivik family alone, on the GPU, against the plain oracle's function for it."""
import pytest
import torch

from oracle import subivik_oracle as oracle
from tests.test_fozerax_ops_gpu import SCAN_SIZES, _close, _cu, _i32, _paged, _rnd, _run_portions, _sequences

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
IDS = ["fp32", "bf16"]
TOL = {torch.float32: 2e-6, torch.bfloat16: 8e-3}
F64 = torch.float64


# ------------------------------------------------------------------------------------------------ norm, stream, mixtures
def _entry(seed, W, dtype, shift=None, alpha=0.6):
    from minivllm_b200.layers.tanh_norm import TanhEntry
    w, b = _rnd(seed, W, dtype=dtype), _rnd(seed + 1, W, dtype=dtype)
    return TanhEntry(torch.tensor(alpha), w.cuda(), b.cuda(), shift), lambda x: oracle.dynamic_tanh(x, alpha, w.double(), b.double())


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width", [91, 64, 2048, 1, 3000, 6160])
def test_stream_steps(width, dtype):
    """The embedding with and without the sinusoids of positions near and far; a sublayer's result; the pieces of a mixture of
    experts; inputs around zero, where tanh is a line, and far out, where it is flat."""
    from minivllm_b200.layers import tanh_norm as TN
    from minivllm_b200.utils.context import reset_context, set_context
    rows, d = 6, lambda t: t.double()
    table, ids = _rnd(1, 11, width, dtype=dtype), torch.tensor([3, 0, 10, 3, 7, 99])
    pos = torch.tensor([0, 1, 77, 511, 8000, -1])
    entry, norm = _entry(10, width, dtype)
    set_context(True, positions=pos.cuda())
    plain = d(table)[ids.clamp_max(10) * (ids < 11)]
    x, h = TN.tanh_embed(ids.cuda(), table.cuda(), entry)
    assert torch.equal(x.cpu(), plain.float())
    _close(h, norm(plain), TOL[dtype], "embedding")
    c = torch.arange(width)
    angle = d(pos)[:, None] * 10000.0 ** (-2.0 * d(c // 2) / width)
    want = plain + torch.where(c % 2 == 1, angle.cos(), angle.sin())
    x, h = TN.tanh_embed(ids.cuda(), table.cuda(), entry, TN.position_frequencies(width, "cuda"))
    _close(x, want, 3e-7, "sinusoids")
    _close(h, norm(want), TOL[dtype], "sinusoids, next input")
    x = _rnd(5, rows, width, scale=2.0)
    x[0], x[1] = x[0] * 1e-3, x[1] * 50
    y = _rnd(2, rows, width + 8, dtype=dtype, scale=0.5)[:, 8:]
    y[0] = y[0] * 1e-3
    want, gx = d(x) + d(y), x.cuda()
    new, h = TN.tanh_step(gx, y.cuda(), entry)
    assert new is gx
    _close(new, want, 3e-7, "result")
    _close(h, norm(want), TOL[dtype], "result, next input")
    flat, zero = _entry(20, width, dtype)[0], torch.zeros(width, dtype=dtype, device="cuda")
    flat.b.data = zero
    small = TN.tanh_step(x[:1].cuda(), y[:1].cuda(), flat)[1]
    _close(small, torch.tanh(0.6 * (d(x) + d(y))[:1]) * d(flat.w.cpu()), TOL[dtype], "around zero")
    for top in (1, 3, 9):
        p = torch.randperm(rows * top, generator=torch.Generator().manual_seed(8)).to(torch.int32).view(rows, top)
        er, tw = _rnd(9, rows * top, width, dtype=dtype), _rnd(10, rows, top)
        want = d(x) + (d(tw)[..., None] * d(er)[p.long()]).sum(1)
        new, h = TN.tanh_step(x.cuda(), (er.cuda(), p.cuda(), tw.cuda()), entry)
        _close(new, want, 5e-7, "experts")
        _close(h, norm(want), TOL[dtype], "experts, next input")
    reset_context()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width,mixes", [(91, 5), (64, 5), (2048, 5), (136, 1), (24, 3)])
@pytest.mark.parametrize("source", ["embedding", "result", "experts"])
def test_token_shift(source, width, mixes, dtype):
    """Mixtures with the token before: single tokens beside portions, cuts everywhere, slots whose old contents must not be
    seen, the first token, a padding row; enough rows that threads begin in the middle of a sequence."""
    from minivllm_b200.layers import tanh_norm as TN
    from minivllm_b200.utils.context import reset_context, set_context
    lens, slots, d = [400, 1, 23, 9], [4, 0, 2, 5], lambda t: t.double()
    shift = TN.TokenShift(torch.rand(mixes, width, generator=torch.Generator().manual_seed(1)).to(dtype).cuda())
    entry, norm = _entry(10, width, dtype, shift)
    table = _rnd(1, 50, width, dtype=dtype)
    ids = [torch.randint(0, 50, (n,), generator=torch.Generator().manual_seed(s)) for s, n in enumerate(lens)]
    ys = [_rnd(20 + s, n, width, dtype=dtype) for s, n in enumerate(lens)]
    ref = []
    for i, y in zip(ids, ys):
        x = d(table)[i]
        x = x if source == "embedding" else x + (d(y) if source == "result" else 0.75 * d(y))
        h = norm(x).to(dtype).double()
        ref.append(torch.stack([oracle.shift_mix(h, d(m.cpu())) for m in shift.mu]))
    for cuts in ([1000], [7, 1, 2, 160], [1], [2, 1]):
        spec, dt = shift.slot_state_spec(dtype)["h"]
        shift.slot_state = {"h": torch.full((7, *spec), float("nan"), dtype=dt, device="cuda")}

        def step(spans):
            spans = sorted(spans, key=lambda x: x[2] - x[1] != 1)
            nd = sum(hi - lo == 1 for _, lo, hi in spans)
            single = nd == len(spans)
            cu = _cu([hi - lo for _, lo, hi in spans])
            set_context(True, None if single else cu, num_decode=nd, portion_cu_q=cu[nd:] - cu[nd],
                        state_slots=_i32([slots[s] for s, _, _ in spans]), state_starts=_i32([lo for _, lo, _ in spans]))
            cat = lambda v: torch.cat([v[s][lo:hi] for s, lo, hi in spans]).cuda()
            want = torch.cat([ref[s][:, lo:hi] for s, lo, hi in spans], 1)
            if source == "embedding":
                _, (h, mixed) = TN.tanh_embed(cat(ids), table.cuda(), entry)
            else:
                x, y = table.cuda()[cat(ids)].float(), cat(ys)
                if source == "experts":
                    rows = torch.arange(len(y), dtype=torch.int32, device="cuda")[:, None]
                    y = (y, rows, torch.full((len(y), 1), 0.75, device="cuda"))
                new, (h, mixed) = TN.tanh_step(x, y, entry)
                assert new is not x
            _close(mixed, want, 2 * TOL[dtype], f"cuts {cuts}, {spans}")

        _run_portions(step, lens, cuts)
        before = shift.slot_state["h"].clone()
        assert bool(before[[1, 3, 6]].isnan().all()) and not bool(before[[4, 0, 2, 5]].isnan().any())
        set_context(False, num_decode=2, state_slots=_i32([6, 6]), state_starts=_i32([-1, -1]))
        TN.tanh_embed(torch.tensor([0, 1]).cuda(), table.cuda(), entry)
        assert torch.equal(shift.slot_state["h"].nan_to_num(7.0), before.nan_to_num(7.0))
    reset_context()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_activations(dtype):
    from minivllm_b200.layers.mlp import xielu
    from minivllm_b200.layers.time_mix import tanh_rows
    for cols in (37, 64, 3000):
        z = _rnd(1, 9, cols + 8, dtype=dtype, scale=3.0)[:, 8:]
        z[0], z[1] = z[0] * 1e-3, z[1] * 0.2
        p, q = torch.tensor(0.4, dtype=F64), torch.tensor(-0.7, dtype=F64)
        a, b = float(oracle.softplus(p)), float(0.5 + oracle.softplus(q))
        got, want = xielu(z.cuda(), a, b), oracle.xielu(z.double(), p, q)
        for r in range(9):               # every row by itself: small inputs too
            _close(got[r], want[r], TOL[dtype], f"xielu, row {r}")
        # what is left beside z / 2 keeps its size near zero
        if dtype == torch.float32:
            curve = (got - z.cuda() / 2).double().cpu()[1]
            _close(curve, (want - z.double() / 2)[1], 1e-5, "curvature")
        _close(tanh_rows(z.float().cuda(), dtype), torch.tanh(z.double()), TOL[dtype], "tanh")


# ------------------------------------------------------------------------------------------------ router, norm per head, store
@pytest.mark.parametrize("experts,top", [(8, 4), (5, 5), (1, 1), (70, 3), (300, 7)])
def test_routing_over_all_experts(experts, top):
    """Weights are probabilities among all experts, not among the chosen, times a factor."""
    from minivllm_b200.layers import moe
    z = _rnd(1, 33, experts, scale=2.0)
    z[0] += 300.0
    idx, weight = moe.route(z.cuda(), None, top, over_all=True, scale=1.7)
    want_idx, want = oracle.route(z.double(), top, 1.7)
    assert torch.equal(idx.cpu().long(), want_idx)
    _close(weight, want, 2e-6)
    kept = moe.route(z.cuda(), None, top, scale=1.7)[1]
    _close(kept, want / want.sum(-1, keepdim=True) * 1.7, 2e-6)
    assert top == experts or float((kept.cpu() - want).abs().max()) > 0.02


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("experts,top,width,ff,tokens", [(5, 2, 72, 40, 33), (8, 4, 64, 128, 200), (3, 1, 90, 21, 10), (4, 4, 136, 72, 3)])
def test_experts(experts, top, width, ff, tokens, dtype):
    from minivllm_b200.layers import moe
    g = {n: _rnd(i, experts, *s, dtype=dtype, scale=s[1] ** -0.5) for i, (n, s) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))))}
    w = {f"e{e}.{n}": t[e] for n, t in g.items() for e in range(experts)}
    w["router"] = _rnd(7, experts, width, dtype=dtype, scale=3.0 * width ** -0.5)
    spec = {"router": {"experts": experts, "top": top, "scale": 1.4}, "expert": {"ff": ff}}
    layer = moe.MixtureOfExperts(spec, width, lambda n, s: w[n].cuda(), router_bias=False, over_all=True)
    h = _rnd(9, tokens, width, dtype=dtype)
    rows, pos, weight = layer.routed(h.cuda())
    got = (weight[..., None].double() * rows.double()[pos.long()]).sum(1)
    _close(got, oracle.moe(h.double(), {k: t.double() for k, t in w.items()}, "", spec), 3 * TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,dim,at", [(3, 10, 5), (4, 64, 64), (1, 40, 12), (16, 128, 8), (2, 256, 0), (2, 1100, 8)])
def test_norm_per_head_into_some_columns(heads, dim, at, dtype):
    from minivllm_b200.layers import group_norm as GN
    n, cols, eps = 7, heads * dim, 1e-3
    y, z, w = (_rnd(i, *s, dtype=dtype) for i, s in enumerate(((n, cols), (n, cols), (cols,))))
    wide = torch.full((n, at + cols + 3), 5.0, dtype=dtype, device="cuda")
    GN.head_norm_gate(y.cuda(), z.cuda(), w.cuda(), heads, eps, out=wide[:, at:at + cols], mult=0.3)
    want = oracle.rms_norm(y.double().view(n, heads, dim), 1.0, eps).view(n, cols) * w.double() * oracle.silu(z.double()) * 0.3
    _close(wide[:, at:at + cols], want, TOL[dtype])
    assert bool((wide[:, :at] == 5).all()) and bool((wide[:, at + cols:] == 5).all())


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,G,VG,d,vd", [(6, 2, 1, 18, 14), (8, 4, 2, 64, 128), (4, 2, 1, 7, 300), (0, 3, 3, 24, 40), (0, 1, 1, 9, 5)])
def test_norm_and_store(H, G, VG, d, vd, dtype):
    """More key heads than value heads; keys and values alone, keys without a norm."""
    from minivllm_b200.layers.rotary_attention import qkv_rope_store
    n, eps, bs = 5, 1e-3, 8
    sizes = (H * d, G * d, VG * vd)
    q, k, v = _rnd(1, n, sum(sizes), dtype=dtype).cuda().split(sizes, 1)
    wq, wk = _rnd(2, d, dtype=dtype), _rnd(3, d, dtype=dtype)
    norm = lambda x, w: oracle.rms_norm(x.double().cpu().view(n, -1, d), w.double(), eps).flatten(1)
    want_q = norm(q, wq) if H else None
    want_k = norm(k, wk) if H else k.double().cpu()
    cache, slots = torch.full((4, bs, G * d + VG * vd), 7.0, dtype=dtype, device="cuda"), torch.tensor([9, -1, 0, 31, 12])
    pos = torch.zeros(n, dtype=torch.int64, device="cuda")
    packed = qkv_rope_store(q if H else None, k, v, wq.cuda() if H else None, wk.cuda() if H else None, None, eps, pos, None, 0, None, H, G,
                            cache, slots.cuda(), packed=True, v_heads=VG)
    _close(packed[:, :G * d], want_k, TOL[dtype], "keys")
    assert torch.equal(packed[:, G * d:], v)
    if H:
        _close(q, want_q, TOL[dtype], "queries")
    flat = cache.view(32, -1)
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(flat[s], packed[i])
    assert bool((flat[[s for s in range(32) if s not in slots.tolist()]] == 7.0).all())


# ------------------------------------------------------------------------------------------------ talking heads
TALK_CASES = [   # heads, kv heads, dim, vdim, cap, block
    (6, 2, 18, 14, 3.0, 16), (6, 3, 64, 128, 18.0, 64), (4, 1, 128, 64, 9.0, 16), (2, 2, 96, 256, 20.0, 8), (20, 1, 40, 24, 30.0, 32),
    (3, 3, 192, 128, 50.0, 16), (1, 1, 8, 8, 20.0, 64), (36, 2, 16, 16, 10.0, 48), (4, 2, 72, 200, 60.0, 16), (16, 8, 128, 64, 15.0, 64),
    (4, 4, 64, 64, 500.0, 16), (5, 5, 24, 72, 20.0, 16)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("case", TALK_CASES, ids=lambda c: "x".join(map(str, c)))
def test_talking_heads(case, dtype):
    """Every kernel form on every token: prompts at once, portions behind cached tokens, single tokens; marked keys near and
    far, at block and tile borders.  One head's bias is steep, one's hardly there."""
    from minivllm_b200.layers import talk_attention as TA
    from minivllm_b200.layers.latent_attention import latent_gather
    H, G, d, vd, cap, bs = case
    lens, tol = [300, 1, 130, 77], 6e-6 if dtype == torch.float32 else 1.2e-2
    scale = 0.35 * cap / d if cap < 100 else 0.8 * d ** -0.5       # a marked key's score is a good part of the cap
    seqs = _sequences(lens, H, G, d, vd, dtype, 3, [0, bs - 1, bs, 63, 64, 127, 128, 200])
    r1, r2 = torch.rand(H, generator=torch.Generator().manual_seed(1)) * 1.5, torch.rand(H, generator=torch.Generator().manual_seed(2)) + 0.05
    r1[0], r1[-1] = 2.5, 0.01
    talk = torch.eye(H) + 0.5 * _rnd(5, H, H)
    full, want = [], []
    for q, k, v in seqs:
        w = oracle.capped_weights(q.double(), k.double(), r1.double(), r2.double(), scale, cap)
        full.append(torch.einsum("gij,jcd->igcd", w, v.double()))
        mixed = oracle.mix_heads(w, talk.double())
        want.append(torch.stack([mixed[h] @ v[:, h // (H // G)].double() for h in range(H)], 1).flatten(1))
    full, want = torch.cat(full), torch.cat(want)
    rows = [torch.cat([k.flatten(1), v.flatten(1)], 1) for _, k, v in seqs]
    cache, tables = _paged(rows, bs, dtype)
    args = (G, d, vd, scale, r1.cuda(), r2.cuda(), cap)
    tiles = dtype == torch.bfloat16 and d % 8 == 0 and vd % 8 == 0 and d <= 128 and cap <= 60
    flat_q = torch.cat([q.flatten(1) for q, _, _ in seqs]).cuda()
    pos, cu = torch.cat([torch.arange(n) for n in lens]).cuda(), _cu(lens)

    def compare(a, sel, what):
        _close(a, full[sel], tol, what)
        out = torch.full((len(sel), H * vd + 8), 3.0, dtype=dtype, device="cuda")
        TA.head_mix(a, talk.cuda(), out[:, 8:], 0.5)
        _close(out[:, 8:], 0.5 * want[sel], tol, what + ", mixed")
        assert bool((out[:, :8] == 3).all())

    every = torch.arange(sum(lens))
    compare(TA.talk_attention_rows(flat_q, cache, tables, cu, pos, *args), every, "rows")
    if tiles:
        packed = torch.cat(rows).cuda()
        compare(TA.talk_prefill(flat_q, packed[:, :G * d], packed[:, G * d:], cu, cu, *args), every, "prefill, whole")
    for part in (2, 31, 76, 129):
        take = [min(part, n) for n in lens]
        sel = torch.cat([torch.arange(n - t, n) + sum(lens[:s]) for s, (n, t) in enumerate(zip(lens, take))])
        cu_q, q, at = _cu(take), flat_q[sel.cuda()], pos[sel.cuda()]
        compare(TA.talk_attention_rows(q, cache, tables, cu_q, at, *args), sel, f"rows, portion of {part}")
        if tiles:
            packed = latent_gather(cache, cu, sum(lens), tables)
            compare(TA.talk_prefill(q, packed[:, :G * d], packed[:, G * d:], cu_q, cu, *args), sel, f"prefill, portion of {part}")
    places = [0, 1, bs - 1, bs, 15, 16, 63, 64, 65, 127, 128, 129, 199, 200, 201, 255, 256, 299]
    for batch in (places, places[-2:]):
        at = torch.tensor(batch).cuda()
        q, tab = flat_q[at], tables[:1].expand(len(batch), -1).contiguous()
        compare(TA.talk_attention_rows(q, cache, tab, None, at, *args), torch.tensor(batch), "rows, one token each")
        out = torch.zeros(len(batch), H * vd + 2, dtype=dtype, device="cuda")
        done = TA.talk_decode(q, cache, tab, at, *args, talk.cuda(), out[:, 2:], 0.5)
        assert done == (dtype == torch.bfloat16 and d % 8 == 0 and vd % 8 == 0 and cap <= 60)
        if done:
            _close(out[:, 2:], 0.5 * want[batch], tol, "decode")
    out = torch.ones(2, H * vd, dtype=dtype, device="cuda")
    if TA.talk_decode(flat_q[:2], cache, torch.full_like(tables[:2], -1), torch.tensor([-1, -1]).cuda(), *args, talk.cuda(), out):
        assert bool((out == 0).all())
    assert int(TA._error_word(flat_q.device).item()) == 0


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_scores_at_the_cap(dtype):
    """Scores far beyond the cap on both sides, from the first token on: the weights stay those of the cap."""
    from minivllm_b200.layers import talk_attention as TA
    H, G, d, vd, bs, n, cap = 4, 2, 64, 64, 16, 150, 60.0
    e = _rnd(1, d)
    sign = torch.where(_rnd(2, n) > 0.8, 1.0, -1.0)
    sign[:20] = -1.0
    q, k, v = e.expand(n, H, d).to(dtype), (e * sign[:, None])[:, None].expand(n, G, d).to(dtype), _rnd(3, n, G, vd, dtype=dtype)
    r1, r2, talk = torch.full((H,), 0.3), torch.full((H,), 0.5), torch.eye(H) + 0.3 * _rnd(4, H, H)
    w = oracle.capped_weights(q.double(), k.double(), r1.double(), r2.double(), 5.0, cap)
    full = torch.einsum("gij,jcd->igcd", w, v.double())
    cache, tables = _paged([torch.cat([k.flatten(1), v.flatten(1)], 1)], bs, dtype)
    args = (G, d, vd, 5.0, r1.cuda(), r2.cuda(), cap)
    pos, cu, flat = torch.arange(n).cuda(), _cu([n]), q.flatten(1).cuda()
    tol = 6e-6 if dtype == torch.float32 else 1.2e-2
    _close(TA.talk_attention_rows(flat, cache, tables, cu, pos, *args), full, tol, "rows")
    if dtype == torch.bfloat16:
        _close(TA.talk_prefill(flat, k.flatten(1).cuda(), v.flatten(1).cuda(), cu, cu, *args), full, tol, "prefill")
        out = torch.empty(n, H * vd, dtype=dtype, device="cuda")
        assert TA.talk_decode(flat, cache, tables.expand(n, -1).contiguous(), pos, *args, talk.cuda(), out)
        mixed = oracle.mix_heads(w, talk.double())
        _close(out, torch.stack([mixed[h] @ v[:, h // 2].double() for h in range(H)], 1).flatten(1), tol, "decode")


@pytest.mark.parametrize("lens", [[2, 3] * 600, [1300, 2, 700, 129, 128, 127, 257]], ids=["many", "long"])
def test_prefill_over_many_units(lens):
    """More sequences than the prefill kernel keeps bounds of, and more units of work than there are SMs; portions behind a past
    of their own.  Against the kernel for any sizes."""
    from minivllm_b200.layers import talk_attention as TA
    H, G, d, vd, bs, cap = 6, 3, 64, 64, 16, 20.0
    behind = [(7 * i) % 40 for i in range(len(lens))]
    total = [n + b for n, b in zip(lens, behind)]
    rows = [_rnd(i, n, G * (d + vd)).bfloat16() for i, n in enumerate(total)]
    q, r1, r2 = 2.0 * _rnd(5, sum(lens), H * d), torch.rand(H).cuda(), torch.rand(H).cuda()
    cache, tables = _paged(rows, bs, torch.bfloat16)
    q, packed = q.bfloat16().cuda(), torch.cat(rows).cuda()
    pos = torch.cat([torch.arange(b, b + n) for n, b in zip(lens, behind)]).cuda()
    args = (G, d, vd, 0.3, r1, r2, cap)
    want = TA.talk_attention_rows(q, cache, tables, _cu(lens), pos, *args)
    got = TA.talk_prefill(q, packed[:, :G * d], packed[:, G * d:], _cu(lens), _cu(total), *args)
    _close(got, want.cpu(), 1.2e-2)
    assert int(TA._error_word(q.device).item()) == 0


def test_a_long_past():
    """One token behind 9,000 others: the only key that matters is the first, the weights reach it past all the others."""
    from minivllm_b200.layers import talk_attention as TA
    H, G, d, vd, bs, n = 8, 2, 64, 64, 64, 9000
    q, k, v = _rnd(1, 1, H * d), 0.05 * _rnd(2, n, G * d), 0.05 * _rnd(3, n, G * vd)
    k[0] = torch.cat([q.view(H, d)[g * 4:(g + 1) * 4].sum(0) for g in range(G)])
    v[0] = 5.0 * _rnd(4, G * vd)
    q, k, v = (t.bfloat16() for t in (q, k, v))
    r1, r2, talk = torch.linspace(0.02, 0.6, H), torch.full((H,), 0.2), torch.eye(H) + 0.3 * _rnd(5, H, H)
    cap, scale = 20.0, 0.4
    kk, s = k.double().view(n, G, d), torch.empty(H, n, dtype=F64)
    for h in range(H):
        x = kk[:, h // 4] @ q.double().view(H, d)[h] * scale
        s[h] = cap * torch.tanh(x / cap) - r1[h].double() * torch.log1p(r2[h].double() * (n - 1 - torch.arange(n)).double())
    w = talk.double() @ torch.softmax(s, -1)
    assert float(w[:, 0].abs().min()) > 0.02
    want = torch.stack([w[h] @ v.double().view(n, G, vd)[:, h // 4] for h in range(H)]).view(1, -1)
    cache, tables = _paged([torch.cat([k, v], 1)], bs, torch.bfloat16)
    args = (G, d, vd, scale, r1.cuda(), r2.cuda(), cap)
    out, at = torch.empty(1, H * vd, dtype=torch.bfloat16, device="cuda"), torch.tensor([n - 1]).cuda()
    assert TA.talk_decode(q.cuda(), cache, tables, at, *args, talk.cuda(), out)
    _close(out, want, 8e-3, "decode")
    rows = torch.cat([k, v], 1).cuda()
    a = TA.talk_prefill(q.cuda(), rows[:, :G * d], rows[:, G * d:], _cu([1]), _cu([n]), *args)
    _close(TA.head_mix(a, talk.cuda(), out), want, 1.2e-2, "prefill")
    a = TA.talk_attention_rows(q.cuda(), cache, tables, None, at, *args)
    _close(TA.head_mix(a, talk.cuda(), out), want, 8e-3, "rows")


# ------------------------------------------------------------------------------------------------ differential attention
DIFF_CASES = [   # heads, kv heads, dim, vdim, chunk, block
    (6, 2, 18, 14, 11, 16), (4, 1, 64, 128, 33, 64), (8, 4, 128, 64, 130, 16), (2, 2, 96, 64, 1, 8), (20, 1, 40, 24, 128, 32),
    (3, 3, 128, 128, 64, 16), (2, 1, 200, 160, 100, 64), (4, 2, 64, 64, 5000, 16), (4, 2, 72, 256, 257, 48), (1, 1, 8, 8, 70, 16),
    (9, 1, 32, 16, 75, 64)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("case", DIFF_CASES, ids=lambda c: "x".join(map(str, c)))
def test_differential_attention(case, dtype):
    """Every kernel form on every token: prompts at once, portions behind cached tokens, single tokens; marked keys at block,
    tile and chunk borders, which the next chunk must not see.  The marked keys of the two maps differ."""
    from minivllm_b200.layers import diff_attention as DA
    from minivllm_b200.layers.latent_attention import latent_gather
    H, G, d, vd, chunk, bs = case
    lens, scale, eps, diff, tol = [300, 1, 130, 77], 0.8 * d ** -0.5, 1e-4, 0.45, 2e-5 if dtype == torch.float32 else 2e-2
    marked = sorted({0, bs - 1, 63, 64, 128, 200, chunk - 1, chunk, 2 * chunk - 1})
    maps = [_sequences(lens, H, G, d, vd, dtype, seed, m) for seed, m in ((3, marked), (4, marked[::2]))]
    vecs = [0.2 * _rnd(20 + i, d) for i in range(4)]
    lam = float(oracle.difference_factor(*(x.double() for x in vecs), diff))
    want, rows, qs, gates = [], [], [], []
    for s, ((q1, k1, v), (q2, k2, _)) in enumerate(zip(*maps)):
        a1, a2 = (oracle.chunk_attention(q.double(), k.double(), v.double(), scale, chunk) for q, k in ((q1, k1), (q2, k2)))
        g = _rnd(60 + s, len(v), H * vd, dtype=dtype)
        o = oracle.rms_norm(a1 - lam * a2, 1.0, eps) * (1 - diff)
        want.append(o.flatten(1) * oracle.sigmoid(g.double()))
        rows.append(torch.cat([torch.stack([k1, k2], 2).flatten(1), v.flatten(1)], 1))
        qs.append(torch.stack([q1, q2], 2).flatten(1))
        gates.append(g)
    cache, tables = _paged(rows, bs, dtype)
    flat_q, gate, want = torch.cat(qs).cuda(), torch.cat(gates).cuda(), torch.cat(want)
    pos, cu = torch.cat([torch.arange(n) for n in lens]).cuda(), _cu(lens)
    even, new = d % 8 == 0 and vd % 8 == 0 and dtype == torch.bfloat16, lambda n: torch.empty(n, H * vd, dtype=dtype, device="cuda")
    tiles = even and d <= 128 and vd <= 128
    end = lambda sel: (chunk, gate[sel], lam, 1 - diff, eps, H, G, d, vd, scale, new(len(sel)))
    every = torch.arange(sum(lens)).cuda()
    _close(DA.diff_attention_rows(flat_q, cache, tables, cu, pos, *end(every)), want, tol, "rows")
    if tiles:
        _close(DA.diff_prefill(flat_q, torch.cat(rows).cuda(), cu, cu, *end(every)), want, tol, "prefill, whole")
    for part in (2, 31, 76, 129):
        take = [min(part, n) for n in lens]
        sel = torch.cat([torch.arange(n - t, n) + sum(lens[:s]) for s, (n, t) in enumerate(zip(lens, take))]).cuda()
        cu_q, ref = _cu(take), want[sel.cpu()]
        _close(DA.diff_attention_rows(flat_q[sel], cache, tables, cu_q, pos[sel], *end(sel)), ref, tol, f"rows, portion of {part}")
        if tiles:
            first = [(n - t) // chunk * chunk for n, t in zip(lens, take)]
            keys = [n - f for n, f in zip(lens, first)]
            packed = latent_gather(cache, _cu(keys), sum(keys), tables, _i32(first))
            _close(DA.diff_prefill(flat_q[sel], packed, cu_q, _cu(keys), *end(sel)), ref, tol, f"prefill, portion of {part}")
    places = sorted({p for m in marked for p in (m - 1, m, m + 1) if 0 <= p < lens[0]} | {p for c in range(0, 300, max(chunk, 37)) for p in (c, c + 1)} | {299})
    for batch in (places, places[-2:]):
        at = torch.tensor(batch).cuda()
        q, tab, ref = flat_q[at], tables[:1].expand(len(batch), -1).contiguous(), want[batch]
        _close(DA.diff_attention_rows(q, cache, tab, None, at, *end(at)), ref, tol, "rows, one token each")
        got = DA.diff_decode(q, cache, tab, at, *end(at))
        assert (got is None) == (not even or d > 128)
        if got is not None:
            _close(got, ref, tol, "decode")
    at = torch.tensor([-1, -1]).cuda()
    got = DA.diff_decode(flat_q[:2], cache, torch.full_like(tables[:2], -1), at, *end(at.clamp_min(0)))
    assert got is None or bool((got == 0).all())
    assert int(DA._error_word(flat_q.device).item()) == 0


def test_maps_that_almost_agree():
    """The first token of a chunk sees itself alone, so that the maps agree and only their factor is left; the norm brings the
    small difference back to size."""
    from minivllm_b200.layers import diff_attention as DA
    H, G, d, vd, chunk, bs, n = 4, 2, 64, 64, 40, 16, 121
    q, v, gate = _rnd(1, n, H * 2 * d).bfloat16(), _rnd(3, n, G, vd).bfloat16(), torch.zeros(n, H * vd, dtype=torch.bfloat16)
    rows = torch.cat([_rnd(2, n, G * 2 * d).bfloat16(), v.flatten(1)], 1)
    cache, tables = _paged([rows], bs, torch.bfloat16)
    firsts = torch.arange(0, n, chunk)
    want = 0.4 * 0.5 * oracle.rms_norm((0.02 * v.double()).repeat_interleave(2, 1), 1.0, 1e-9)[firsts].flatten(1)
    end = lambda m: (chunk, gate[:m].cuda(), 0.98, 0.4, 1e-9, H, G, d, vd, 0.3, torch.empty(m, H * vd, dtype=torch.bfloat16, device="cuda"))
    pos, cu = torch.arange(n).cuda(), _cu([n])
    for got in (DA.diff_prefill(q.cuda(), rows.cuda(), cu, cu, *end(n))[firsts.cuda()],
                DA.diff_attention_rows(q.cuda(), cache, tables, cu, pos, *end(n))[firsts.cuda()],
                DA.diff_decode(q[firsts].cuda(), cache, tables.expand(len(firsts), -1).contiguous(), firsts.cuda(), *end(len(firsts)))):
        _close(got, want, 8e-3)


# ------------------------------------------------------------------------------------------------ time mixing
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,K,V", SCAN_SIZES)
def test_time_scan(heads, K, V, dtype):
    """Portions and single tokens from slots whose old contents must not be seen; channels that forget at once beside channels
    that never do; a bonus of both signs."""
    from minivllm_b200.layers import time_mix as L
    lens, eps, d = [70, 1, 33], 1e-4, lambda t: t.double()
    w0, bonus, w = _rnd(70, heads * K, dtype=dtype), _rnd(71, heads, K, dtype=dtype), _rnd(77, heads * V, dtype=dtype)
    seqs, ref = [], []
    for s, n in enumerate(lens):
        q, k, v, g = (_rnd(10 * s + i, n, heads, D, dtype=dtype) for i, D in enumerate((K, K, V, V)))
        z = _rnd(10 * s + 5, n, heads, K, scale=2.0) - 2.0
        z[:, :, 0], z[:, :, -1] = 60.0, -30.0
        seqs.append((q, k, v, g, z))
        ref.append(oracle.bonus_scan(d(q), d(k), d(v), torch.exp(-torch.exp(d(z) + d(w0).view(heads, K))), d(bonus)))
    gated = [(oracle.rms_norm(o, 1.0, eps).flatten(1) * d(w) * oracle.silu(d(x[3])).flatten(1)) * 0.6 for (o, _), x in zip(ref, seqs)]
    slots, tol = [4, 0, 2], 3e-6 if dtype == torch.float32 else 6e-3
    for cuts in ([100], [7, 1, 2, 16], [1]):
        state = torch.full((6, heads, K, V), float("nan"), device="cuda")

        def step(spans):
            cat = lambda i: torch.cat([seqs[s][i][a:b].flatten(1) for s, a, b in spans])
            q, k, v, g = torch.cat([cat(0), cat(1), cat(2), cat(3)], 1).cuda().split([heads * K, heads * K, heads * V, heads * V], 1)
            sl, st = _i32([slots[s] for s, _, _ in spans]), _i32([a for _, a, _ in spans])
            single = all(b - a == 1 for _, a, b in spans)
            cu = None if single else _cu([b - a for _, a, b in spans])
            got = L.time_scan(q, k, v, cat(4).cuda(), w0.cuda(), bonus.cuda(), cu, sl, st, state, heads, K, V, gate=g, norm_w=w.cuda(),
                              eps=eps, out_scale=0.6)
            want = torch.cat([(gated[s] if single else ref[s][0].flatten(1))[a:b] for s, a, b in spans])
            _close(got, want, tol * (3 if single else 1), f"cuts {cuts}, {spans}")

        _run_portions(step, lens, cuts)
        for s in range(len(lens)):
            _close(state[slots[s]], ref[s][1], 3e-6 if dtype == torch.float32 else 1e-4, "state")
        assert bool(state[[1, 3, 5]].isnan().all())


@pytest.mark.parametrize("K,V", [(64, 64), (128, 128), (32, 24), (96, 72), (48, 48), (8, 200)])
def test_chunked_time_scan(K, V):
    """The chunked kernels on portions cut inside and at the edges of chunks and blocks: decays from none to complete within a
    block, an entry read out by its own token alone, and the token after the last of a chunk."""
    from minivllm_b200.layers import time_mix as L
    heads, lens, d = 3, [200, 64, 65, 17], lambda t: t.double()
    w0, bonus = _rnd(1, heads * K).bfloat16(), (2.0 * _rnd(2, heads, K)).bfloat16()
    seqs, ref = [], []
    for s, n in enumerate(lens):
        q, k, v = (_rnd(10 * s + i, n, heads, D).bfloat16() for i, D in enumerate((K, K, V)))
        z = _rnd(10 * s + 5, n, heads, K, scale=1.5) - 3.0
        z[:, 1] = _rnd(10 * s + 6, n, K, scale=3.0)           # a head that forgets more than a block's factors can hold
        z[n // 2, 2] = 5.0                                    # one token clears a head's past
        seqs.append((q, k, v, z))
        ref.append(oracle.bonus_scan(d(q), d(k), d(v), torch.exp(-torch.exp(d(z) + d(w0).view(heads, K))), d(bonus)))
    slots = [2, 0, 3, 1]
    for cuts in ([1000], [64], [16, 48, 65], [33, 100, 20]):
        state = torch.full((4, heads, K, V), float("nan"), device="cuda")

        def step(spans):
            cat = lambda i: torch.cat([seqs[s][i][a:b].flatten(1) for s, a, b in spans])
            q, k, v = torch.cat([cat(0), cat(1), cat(2)], 1).cuda().split([heads * K, heads * K, heads * V], 1)
            got = L.time_scan(q, k, v, cat(3).cuda(), w0.cuda(), bonus.cuda(), _cu([b - a for _, a, b in spans]),
                              _i32([slots[s] for s, _, _ in spans]), _i32([a for _, a, _ in spans]), state, heads, K, V, chunked=True)
            _close(got, torch.cat([ref[s][0].flatten(1)[a:b] for s, a, b in spans]), 6e-3, f"cuts {cuts}, {spans}")

        _run_portions(step, lens, cuts)
        for s in range(len(lens)):
            _close(state[slots[s]], ref[s][1], 2e-4, "state")


def test_padding_rows_leave_the_state_alone():
    from minivllm_b200.layers import time_mix as L
    H, K = 2, 32
    state, x = _rnd(1, 3, H, K, K).cuda(), _rnd(2, 2, 4 * H * K).cuda()
    before, z = state.clone(), torch.zeros(2, H * K, device="cuda")
    r, k, v, g = x.split(H * K, 1)
    one = torch.ones(H * K, device="cuda")
    out = L.time_scan(r, k, v, z, one, one.view(H, K), None, _i32([2, 2]), _i32([-1, -1]), state, H, K, K, gate=g, norm_w=one)
    assert torch.equal(state, before) and bool((out == 0).all())


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_an_entry_read_out_thousands_of_tokens_later(dtype):
    """Slow decays: the first token's entry is most of what the last token reads; whole, in portions, token by token at the end."""
    from minivllm_b200.layers import time_mix as L
    H, K, n = 1, 64, 3000
    q, k, v = 0.02 * _rnd(1, n, K), 0.02 * _rnd(2, n, K), 0.02 * _rnd(3, n, K)
    k[0] = q[-1] = _rnd(4, K)
    v[0] = _rnd(5, K)
    z = torch.full((n, K), -8.0) + 0.3 * _rnd(6, n, K)
    q, k, v = (t.to(dtype) for t in (q, k, v))
    zero, bonus = torch.zeros(K, dtype=dtype), torch.zeros(1, K, dtype=dtype)
    d = lambda t: t.double()[:, None]
    want, S = oracle.bonus_scan(d(q), d(k), d(v), torch.exp(-torch.exp(d(z))), bonus.double())
    for cuts in ([n], [1000, 999, 64, 1], [2500] + [1] * 500):
        state, at, out, cuts = torch.full((1, 1, K, K), float("nan"), device="cuda"), 0, [], cuts + [n]
        for c in cuts:
            c = min(c, n - at)
            if not c:
                break
            sl = slice(at, at + c)
            p = torch.cat([q[sl], k[sl], v[sl]], 1).cuda().split(K, 1)
            out.append(L.time_scan(*p, z[sl].cuda(), zero.cuda(), bonus.cuda(), _cu([c]), _i32([0]), _i32([at]), state, H, K, K))
            at += c
        _close(torch.cat(out)[-1:], want[-1:].flatten(1), 2e-5 if dtype == torch.float32 else 8e-3, f"{cuts[:3]}")
        _close(state[0], S, 5e-5 if dtype == torch.float32 else 5e-4, "state")
