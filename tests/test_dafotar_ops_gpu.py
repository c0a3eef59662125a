"""Every mechanism of the Dafotar family alone, on the GPU, against the plain oracle's function for it."""
import pytest
import torch

from oracle import dafotar_oracle as oracle
from tests.test_fozerax_ops_gpu import SCAN_SIZES, _close, _cu, _i32, _paged, _rnd, _run_portions

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
IDS = ["fp32", "bf16"]
TOL = {torch.float32: 3e-6, torch.bfloat16: 8e-3}


# ------------------------------------------------------------------------------------------------ streams
def _entry(seed, W, S, dtype, bias=True, conv=None, eps=1e-4):
    from minivllm_b200.layers.streams import StreamEntry
    v = [_rnd(seed, S, dtype=dtype), _rnd(seed + 1, W, dtype=dtype), _rnd(seed + 2, W, dtype=dtype) if bias else None]
    return v, StreamEntry(*(t.cuda() if t is not None else None for t in v), eps, conv)


def _norm(u, w, b, eps):
    return oracle.layer_norm(u, w.double(), b.double(), eps) if b is not None else oracle.rms_norm(u, w.double(), eps)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("width", [90, 64, 2048, 3000, 41, 7168, 9000])
def test_stream_steps(width, S, dtype):
    """The embedding in all streams, a sublayer's result in all streams, the sum in front of the head; layer norm and RMS
    norm."""
    from minivllm_b200.layers import streams as ST
    rows, eps, d = 5, 1e-4, lambda t: t.double()
    table, ids = _rnd(1, 11, width, dtype=dtype), torch.tensor([3, 0, 10, 3, 7])
    y = _rnd(2, rows, width + 8, dtype=dtype, scale=2.0)[:, 8:]
    mix, out = _rnd(3, S, S, dtype=dtype), _rnd(4, S, dtype=dtype)
    for bias in (True, False):
        (a, w, b), entry = _entry(10, width, S, dtype, bias)
        x, h = ST.stream_embed(ids.cuda(), table.cuda(), S, entry)
        want = d(table)[ids].expand(S, -1, -1)
        assert torch.equal(x.cpu(), want.transpose(0, 1).float())
        _close(h, _norm(oracle.gather_streams(want, d(a)), w, b, eps), TOL[dtype], "embedding")
        x = _rnd(5, rows, S, width, scale=1.5) + 0.7
        want = oracle.update_streams(d(x).transpose(0, 1), d(y), d(mix), d(out))
        gx = x.cuda()
        h = ST.stream_step(gx, y.cuda(), mix.cuda(), out.cuda(), entry)
        _close(gx, want.transpose(0, 1), 1e-6, "streams")
        _close(h, _norm(oracle.gather_streams(want, d(a)), w, b, eps), TOL[dtype], "next input")
        entry.w_in = None
        h = ST.stream_step(x.cuda(), y.cuda(), mix.cuda(), out.cuda(), entry)
        _close(h, _norm(want.sum(0), w, b, eps), TOL[dtype], "sum")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width,taps,S", [(90, 4, 3), (64, 1, 2), (2048, 3, 2), (41, 2, 1), (256, 4, 4), (136, 6, 2), (4096, 2, 1),
                                          (24, 5, 5), (512, 9, 3)])
def test_input_convolution(width, taps, S, dtype):
    """Single tokens beside portions, cuts everywhere, slots whose old contents must not be seen; a padding row."""
    from minivllm_b200.layers import streams as ST
    from minivllm_b200.utils.context import reset_context, set_context
    lens, slots, eps, d = [40, 1, 23, 9], [4, 0, 2, 5], 1e-4, lambda t: t.double()
    table = _rnd(1, 50, width, dtype=dtype)
    ids = [torch.randint(0, 50, (n,), generator=torch.Generator().manual_seed(s)) for s, n in enumerate(lens)]
    conv = ST.InputConvolution(_rnd(2, width, taps, dtype=dtype).cuda())
    (a, w, b), entry = _entry(10, width, S, dtype, conv=conv)
    ref = []
    for i in ids:
        h = _norm(d(table)[i] * d(a).sum(), w, b, eps).to(dtype).double()
        ref.append(h + oracle.causal_conv(h, d(conv.weight.cpu())))
    for cuts in ([100], [7, 1, 2, 16], [1], [2, 1]):
        spec, dt = conv.slot_state_spec(dtype)["h"]
        conv.slot_state = {"h": torch.full((7, *spec), float("nan"), dtype=dt, device="cuda")}

        def step(spans):
            spans = sorted(spans, key=lambda x: x[2] - x[1] != 1)
            nd = sum(hi - lo == 1 for _, lo, hi in spans)
            cu = _cu([hi - lo for _, lo, hi in spans])
            set_context(True, cu, num_decode=nd, portion_cu_q=cu[nd:] - cu[nd],
                        state_slots=_i32([slots[s] for s, _, _ in spans]), state_starts=_i32([lo for _, lo, _ in spans]))
            _, h = ST.stream_embed(torch.cat([ids[s][lo:hi] for s, lo, hi in spans]).cuda(), table.cuda(), S, entry)
            want = torch.cat([ref[s][lo:hi] for s, lo, hi in spans])
            _close(h, want, 4 * TOL[dtype], f"cuts {cuts}, {spans}")
            if dtype == torch.float32:
                _close(h, want, 3e-6, f"cuts {cuts}, {spans}")

        _run_portions(step, lens, cuts)
        before = conv.slot_state["h"].clone()
        assert taps == 1 or bool(before[[1, 3, 6]].isnan().all())
        set_context(False, num_decode=2, state_slots=_i32([6, 6]), state_starts=_i32([-1, -1]))
        ST.stream_embed(torch.tensor([0, 1]).cuda(), table.cuda(), S, entry)
        assert torch.equal(conv.slot_state["h"].nan_to_num(7.0), before.nan_to_num(7.0))
    reset_context()


# ------------------------------------------------------------------------------------------------ attention
def _pairs(x, dims):
    """Columns of every head (.., d) in the order in which rotated pairs are neighbours."""
    from minivllm_b200.layers.rotary_attention import pair_order
    return x[..., pair_order(x.shape[-1], dims)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,G,d,vd,dims", [(6, 2, 18, 14, 12), (4, 4, 64, 64, 64), (16, 4, 128, 128, 128), (3, 1, 7, 2, 0), (8, 2, 128, 64, 20),
                                           (2, 1, 200, 160, 200), (2, 2, 40, 256, 36), (1, 1, 520, 24, 8), (5, 1, 33, 300, 2), (2, 1, 8, 8, 8)])
def test_norm_rotation_and_store(H, G, d, vd, dims, dtype):
    from minivllm_b200.layers import rotary_attention as RA
    from minivllm_b200.layers.latent_attention import rope_table
    eps, base, n, bs = 1e-3, 50.0, 5, 8
    pos = torch.tensor([0, 1, 77, 500, 3])
    sizes = (H * d, G * d, G * vd)
    pad = [-s % 8 for s in sizes]
    p = _rnd(1, n, sum(sizes) + sum(pad), dtype=dtype)
    cut = lambda t: (t[:, :sizes[0]], t[:, sizes[0] + pad[0]:][:, :sizes[1]], t[:, sizes[0] + pad[0] + sizes[1] + pad[1]:][:, :sizes[2]])
    q, k, v = (t.double().view(n, -1, e) for t, e in zip(cut(p), (d, d, vd)))
    wq, wk, temp = _rnd(2, d, dtype=dtype), _rnd(3, d, dtype=dtype), _rnd(4, H, dtype=dtype)
    turned = lambda x, w: oracle.rotate(oracle.rms_norm(x, w.double(), eps), pos.double(), base, dims)
    want_q = _pairs(turned(q, wq) * temp.double()[:, None], dims).reshape(n, -1)
    want = torch.cat([_pairs(turned(k, wk), dims).reshape(n, -1), _pairs(oracle.rotate(v, pos.double(), base, vd), vd).reshape(n, -1)], 1)
    # the kernel works on reordered columns
    g = torch.zeros_like(p)
    for dst, src, e in zip(cut(g), (q, k, v), (dims, dims, vd)):
        dst.copy_(_pairs(src, e).reshape(n, -1))
    g = g.cuda()
    table = rope_table(base, dims, 512, "cuda") if dims else None
    cache, slots = torch.full((4, bs, G * (d + vd)), 7.0, dtype=dtype, device="cuda"), torch.tensor([9, -1, 0, 31, 12])
    gq, gk, gv = cut(g.clone())
    args = (_pairs(wq, dims).cuda(), _pairs(wk, dims).cuda(), temp.cuda(), eps, pos.cuda(), table, dims)
    packed = RA.qkv_rope_store(gq, gk, gv, *args, rope_table(base, vd, 512, "cuda"), H, G, cache, slots.cuda(), packed=True)
    _close(gq, want_q, TOL[dtype], "queries")
    _close(packed, want, TOL[dtype], "keys and values")
    flat = cache.view(32, -1)
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(flat[s], packed[i])
    assert bool((flat[[s for s in range(32) if s not in slots.tolist()]] == 7.0).all())
    # queries alone, values as they are
    only = cut(g.clone())[0]
    assert RA.qkv_rope_store(only, None, None, *args, None, H, G) is None
    assert torch.equal(only, gq)
    gq, gk, gv = cut(g.clone())
    plain = RA.qkv_rope_store(gq, gk, gv, *args[:2], None, *args[3:], None, H, G, packed=True)
    assert torch.equal(plain[:, G * d:], gv)
    _close(gq, _pairs(turned(q, wq), dims).reshape(n, -1), TOL[dtype], "without a factor")


WINDOW_CASES = [   # heads, kv heads, dim, vdim, window, block
    (6, 2, 18, 14, 11, 16), (4, 1, 64, 128, 33, 64), (8, 4, 128, 64, 130, 16), (2, 2, 96, 64, 1, 8), (20, 1, 40, 24, 128, 32),
    (3, 3, 192, 128, 64, 16), (2, 1, 200, 160, 100, 64), (4, 2, 64, 64, 5000, 16), (4, 2, 136, 72, 257, 48), (2, 1, 24, 96, 75, 64),
    (1, 1, 8, 8, 70, 16), (2, 2, 64, 256, 40, 16)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("case", WINDOW_CASES, ids=lambda c: "x".join(map(str, c)))
def test_window_attention_with_rotated_values(case, dtype):
    """Every kernel form on every token: prompts at once, portions behind cached tokens, single tokens; marked keys at block
    and tile borders, seen up to exactly one window later; values turned by their positions and results turned back."""
    from minivllm_b200.layers import window_attention as WA
    from minivllm_b200.layers.latent_attention import latent_gather
    from minivllm_b200.layers.rotary_attention import turn_table
    from tests.test_fozerax_ops_gpu import _sequences
    H, G, d, vd, window, bs = case
    lens, scale, base, tol = [300, 1, 130, 77], 0.8 * d ** -0.5, 700.0, 1e-5 if dtype == torch.float32 else 1.6e-2
    marked = [0, bs - 1, bs, 63, 64, 127, 128, 200]
    seqs = _sequences(lens, H, G, d, vd, dtype, 3, marked)
    want, rows = [], []
    for q, k, v in seqs:
        pos = torch.arange(len(q)).double()
        v = oracle.rotate(v.double(), pos, base, vd).to(dtype)
        o = oracle.windowed_attention(q.double(), k.double(), v.double(), torch.full((H,), scale, dtype=torch.float64), window)
        want.append(_pairs(oracle.rotate(o, -pos, base, vd), vd).flatten(1))
        rows.append(torch.cat([k.flatten(1), _pairs(v, vd).flatten(1)], 1))
    cache, tables = _paged(rows, bs, dtype)
    args, kw = (G, d, vd, window, scale), {"turn": turn_table(base, vd, 310, "cuda")}
    tiles = dtype == torch.bfloat16 and d % 8 == 0 and vd % 8 == 0 and d <= 192 and vd <= 128
    flat_q, flat_want = torch.cat([q.flatten(1) for q, _, _ in seqs]).cuda(), torch.cat(want)
    pos = torch.cat([torch.arange(n) for n in lens]).cuda()
    cu = _cu(lens)
    _close(WA.window_attention_rows(flat_q, cache, tables, cu, pos, *args, **kw), flat_want, tol, "rows")
    if tiles:
        _close(WA.window_prefill(flat_q, torch.cat(rows).cuda(), cu, cu, *args, positions=pos, **kw), flat_want, tol, "prefill, whole")
    for part in (2, 31, 76):
        take = [min(part, n) for n in lens]
        sel = torch.cat([torch.arange(n - t, n) + sum(lens[:s]) for s, (n, t) in enumerate(zip(lens, take))]).cuda()
        cu_q, ref = _cu(take), flat_want[sel.cpu()]
        _close(WA.window_attention_rows(flat_q[sel], cache, tables, cu_q, pos[sel], *args, **kw), ref, tol, f"rows, portion of {part}")
        if tiles:
            first = [max(0, n - t - window + 1) for n, t in zip(lens, take)]
            keys = [n - f for n, f in zip(lens, first)]
            packed = latent_gather(cache, _cu(keys), sum(keys), tables, _i32(first))
            got = WA.window_prefill(flat_q[sel], packed, cu_q, _cu(keys), *args, positions=pos[sel], **kw)
            _close(got, ref, tol, f"prefill, portion of {part}")
    places = sorted({p for m in marked for p in (m, m + 1, m + window - 1, m + window) if p < lens[0]} | {299})
    for batch in (places, places[-2:]):
        at = torch.tensor(batch).cuda()
        q, tab, ref = flat_q[at], tables[:1].expand(len(batch), -1).contiguous(), flat_want[batch]
        _close(WA.window_attention_rows(q, cache, tab, None, at, *args, **kw), ref, tol, "rows, one token each")
        got = WA.window_decode(q, cache, tab, at, *args, **kw)
        assert (got is None) == (dtype == torch.float32 or bool(d % 8 or vd % 8))
        if got is not None:
            _close(got, ref, tol, "decode")
    got = WA.window_decode(flat_q[:2], cache, torch.full_like(tables[:2], -1), torch.tensor([-1, -1]).cuda(), *args, **kw)
    assert got is None or bool((got == 0).all())
    assert int(WA._error_word(flat_q.device).item()) == 0


def test_a_common_shift_of_positions_changes_nothing():
    """Keys, values and results depend on distances only: the same rows at later positions give the same results."""
    from minivllm_b200.layers import rotary_attention as RA
    from minivllm_b200.layers import window_attention as WA
    from minivllm_b200.layers.latent_attention import rope_table
    H, G, d, vd, n = 4, 2, 64, 32, 90
    p = _rnd(1, n, H * d + G * (d + vd)).cuda()
    table, vtable = rope_table(1e3, d, 2000, "cuda"), rope_table(1e3, vd, 2000, "cuda")
    one, turn, outs = torch.ones(d, device="cuda"), RA.turn_table(1e3, vd, 2000, "cuda"), []
    for shift in (0, 64, 1024):
        q, k, v = p.clone().split([H * d, G * d, G * vd], 1)
        cache = torch.zeros(24, 64, G * (d + vd), device="cuda")
        pos = torch.arange(n, device="cuda") + shift
        tab = torch.arange(24, dtype=torch.int32, device="cuda")[None]
        RA.qkv_rope_store(q, k, v, one, one, None, 1e-5, pos, table, d, vtable, H, G, cache, pos)
        outs.append(WA.window_attention_rows(q.contiguous(), cache, tab, _cu([n]), pos, G, d, vd, 30, 0.3, turn=turn))
        plain = WA.window_attention_rows(q.contiguous(), cache, tab, _cu([n]), pos, G, d, vd, 30, 0.3)
        assert float((plain - outs[-1]).abs().max()) > 0.1
    # from the first token on whose window lies behind the shift
    _close(outs[1][29:], outs[0][29:].cpu(), 2e-5, "shifted by 64")
    _close(outs[2][29:], outs[0][29:].cpu(), 5e-5, "shifted by 1024")


# ------------------------------------------------------------------------------------------------ matrix memory
def _gates(seed, n, H, cap):
    """Logits and biases; the last head's input gate rises and falls by most of the cap, the first head's forget gate shuts
    now and then."""
    z = _rnd(seed, n, 2 * H, scale=2.0)
    z[:, H:] += 3.0
    z[:, H - 1] += 0.8 * cap * torch.sin(torch.arange(n) / 9.0)
    z[::11, H] = -2.0 * cap
    return z


def _memory_refs(seqs, H, K, V, i_b, f_b, cap):
    out = []
    for q, k, v, _, z in seqs:
        i = oracle.soft_cap(z[:, :H].double() + i_b.double(), cap)
        f = oracle.log_sigmoid(oracle.soft_cap(z[:, H:].double() + f_b.double(), cap))
        out.append(oracle.mlstm_scan(q.double() * K ** -0.5, k.double(), v.double(), i, f) + (i, f))
    return out


def _as_product(z, dtype):
    """An input and weights whose product are the logits z: every logit in four terms of the type."""
    terms, left = [], z.cuda().double()
    for _ in range(4):
        terms.append(left.to(dtype))
        left = left - terms[-1].double()
    return torch.cat(terms, 1), torch.eye(z.shape[1], dtype=dtype, device="cuda").repeat(1, 4)


def _poison(slots, H, K, V):
    return tuple(torch.full((slots, *s), float("nan"), device="cuda") for s in ((H, K, V), (H, K), (H,)))


def _check_state(got, want, slot, tol, tol_m=1e-5):
    """S and n without their common scale, which takes up the rounding of m, and m."""
    shift = torch.exp(got[2][slot].cpu().double() - want[2])
    _close(got[0][slot].cpu().double() * shift[:, None, None], want[0], tol, "S")
    _close(got[1][slot].cpu().double() * shift[:, None], want[1], tol, "n")
    assert float((shift - 1.0).abs().max()) < tol_m


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,K,V", SCAN_SIZES)
def test_mlstm_scan_and_step(H, K, V, dtype):
    """Portions and single tokens, token by token, from slots whose old contents must not be seen."""
    from minivllm_b200.layers import group_norm as GN
    from minivllm_b200.layers import mlstm as L
    lens, cap, eps = [70, 1, 33], 6.0, 1e-4
    seqs = [tuple(_rnd(10 * s + i, n, H, D, dtype=dtype) for i, D in enumerate((K, K, V, V))) + (_gates(10 * s + 7, n, H, cap),)
            for s, n in enumerate(lens)]
    i_b, f_b, w = _rnd(71, H, dtype=dtype), _rnd(72, H, dtype=dtype), _rnd(73, H * V, dtype=dtype)
    ref = _memory_refs(seqs, H, K, V, i_b, f_b, cap)
    gated = [oracle.rms_norm(r[0], 1.0, eps).flatten(1) * w.double() * oracle.sigmoid(x[3].double().flatten(1)) for r, x in zip(ref, seqs)]
    slots, tol = [4, 0, 2], 5e-5 if dtype == torch.float32 else 1.2e-2
    for cuts in ([100], [7, 1, 2, 16], [1]):
        state = _poison(6, H, K, V)

        def step(spans):
            cat = lambda i: torch.cat([seqs[s][i][a:b].flatten(1) for s, a, b in spans])
            p = torch.cat([cat(0), cat(1), cat(2), cat(3)], 1).cuda()
            q, k, v, g = p.split([H * K, H * K, H * V, H * V], 1)
            z, sl, st = cat(4).cuda(), _i32([slots[s] for s, _, _ in spans]), _i32([a for _, a, _ in spans])
            if all(b - a == 1 for _, a, b in spans):
                got = L.mlstm_step(q, k, v, *_as_product(z, dtype), i_b.cuda(), f_b.cuda(), cap, sl, st, *state, H, K, V, g, w.cuda(), eps)
            else:
                cu = _cu([b - a for _, a, b in spans])
                chain = L.mlstm_gates(z, i_b.cuda(), f_b.cuda(), cap, cu, sl, st, state[2], H)
                for col in (0, 1):
                    _close(chain[..., col], torch.cat([ref[s][2 + col][a:b] for s, a, b in spans]), 1e-5, "gates")
                o, den = L.mlstm_scan(q, k, v, chain, cu, sl, st, *state[:2], H, K, V, chunked=False)
                read = o.view(-1, H, V).double().cpu() / den.double().cpu()[..., None]
                _close(read, torch.cat([ref[s][0][a:b] for s, a, b in spans]), tol, f"read-outs, cuts {cuts}, {spans}")
                got = GN.head_norm_gate(o, g, w.cuda(), H, eps, den=den, act="sigmoid")
            _close(got, torch.cat([gated[s][a:b] for s, a, b in spans]), tol, f"cuts {cuts}, {spans}")

        _run_portions(step, lens, cuts)
        for s in range(len(lens)):
            _check_state(state, ref[s][1], slots[s], 2e-5)
        assert all(bool(t[[1, 3, 5]].isnan().all()) for t in state)


@pytest.mark.parametrize("K,V", [(64, 64), (128, 128), (32, 24), (96, 72), (128, 256), (8, 200), (48, 64)])
def test_mlstm_chunks(K, V):
    """The chunked kernels against the oracle: lengths around the chunk size, cuts inside chunks, one sequence and several,
    gates that shut and open; nothing of the state is rounded to 16 bits."""
    from minivllm_b200.layers import mlstm as L
    bf, H, cap = torch.bfloat16, 2, 11.0
    i_b, f_b = torch.tensor([0.5, -1.0]).to(bf), torch.tensor([1.0, 4.0]).to(bf)
    for lens in ([1, 63, 64, 65, 130, 2], [300]):
        seqs = [tuple(_rnd(10 * s + i, n, H, D).to(bf) for i, D in enumerate((K, K, V))) + (None, _gates(10 * s + 7, n, H, cap))
                for s, n in enumerate(lens)]
        ref = _memory_refs(seqs, H, K, V, i_b, f_b, cap)
        for cuts in ([400], [70, 3, 64, 1], [37]):
            state = _poison(len(lens), H, K, V)

            def step(spans):
                cat = lambda i: torch.cat([seqs[s][i][a:b].flatten(1) for s, a, b in spans]).cuda()
                sl, st, cu = _i32([s for s, _, _ in spans]), _i32([a for _, a, _ in spans]), _cu([b - a for _, a, b in spans])
                q, k, v = torch.cat([cat(0), cat(1), cat(2)], 1).split([H * K, H * K, H * V], 1)
                chain = L.mlstm_gates(cat(4), i_b.cuda(), f_b.cuda(), cap, cu, sl, st, state[2], H)
                o, den = L.mlstm_scan(q, k, v, chain, cu, sl, st, *state[:2], H, K, V, chunked=True)
                read = o.view(-1, H, V).double().cpu() / den.double().cpu()[..., None]
                _close(read, torch.cat([ref[s][0][a:b] for s, a, b in spans]), 6e-3, f"{lens}, {spans}")

            _run_portions(step, lens, cuts)
            for s in range(len(lens)):
                _check_state(state, ref[s][1], s, 1e-4)


def test_the_maximum_starts_at_zero():
    """With input gates far below zero the first tokens divide by exp(-m) of a maximum that came from zero."""
    from minivllm_b200.layers import mlstm as L
    H, K, V, n, cap = 1, 8, 4, 12, 20.0
    q, k, v = (_rnd(i, n, H, D) for i, D in enumerate((K, K, V)))
    z = torch.cat([torch.full((n, H), -14.0), torch.full((n, H), -0.5)], 1)
    zero = torch.zeros(H)
    (o, last, i, f), = _memory_refs([(q, k, v, None, z)], H, K, V, zero, zero, cap)
    wrong, m = [], -float("inf")
    for t in range(n):
        m = max(float(f[t, 0]) + m, float(i[t, 0]))
        wrong.append(m)
    assert abs(wrong[0] - float(f[0, 0])) > 5                 # a maximum from minus infinity would differ
    state = _poison(1, H, K, V)
    p = torch.cat([q, k, v], 2).flatten(1).cuda()
    args = (zero.cuda(), zero.cuda(), cap, _cu([n]), _i32([0]), _i32([0]))
    chain = L.mlstm_gates(z.cuda(), *args, state[2], H)
    qs, ks, vs = p.split([K, K, V], 1)
    out, den = L.mlstm_scan(qs, ks, vs, chain, *args[3:], *state[:2], H, K, V)
    _close(out / den, o[:, 0], 2e-5, "read-outs")
    state2, rows = _poison(1, H, K, V), []
    for t in range(n):
        g, w = torch.full((1, V), 40.0, device="cuda"), torch.ones(V, device="cuda")
        rows.append(L.mlstm_step(qs[t:t + 1], ks[t:t + 1], vs[t:t + 1], *_as_product(z[t:t + 1], torch.float32), *args[:3], _i32([0]), _i32([t]), *state2, H, K, V,
                                 g, w, 1e-12))
    _close(torch.cat(rows), oracle.rms_norm(o, 1.0, 1e-12)[:, 0], 2e-5, "steps")
    _check_state(state2, last, 0, 2e-5)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,width", [(1, 2048), (3, 90), (5, 4104), (2, 8)])
def test_gate_logits_of_a_step(H, width, dtype):
    """The product inside the one-token step: any width, rows of a wider tensor."""
    from minivllm_b200.layers import mlstm as L
    K, V, B, cap = 8, 12, 3, 5.0
    x, gw = _rnd(1, B, width + 8, dtype=dtype)[:, 8:], _rnd(2, 2 * H, width, dtype=dtype, scale=2.0 * width ** -0.5)
    q, k, v, g = (_rnd(3 + i, B, H * D, dtype=dtype) for i, D in enumerate((K, K, V, V)))
    b = _rnd(8, H, dtype=dtype)
    state = _poison(B, H, K, V)
    p = torch.cat([q, k, v, g], 1).cuda().split([H * K, H * K, H * V, H * V], 1)
    L.mlstm_step(*p[:3], x.cuda(), gw.cuda(), b.cuda(), b.cuda(), cap, _i32([2, 0, 1]), _i32([0, 0, 0]), *state, H, K, V, p[3],
                 torch.ones(H * V, dtype=dtype, device="cuda"), 1e-6)
    z = x.double() @ gw.double().t()
    i = oracle.soft_cap(z[:, :H] + b.double(), cap)
    f = oracle.log_sigmoid(oracle.soft_cap(z[:, H:] + b.double(), cap))
    m = torch.maximum(f, i)
    _close(state[2][[2, 0, 1]], m, 3e-6, "maximum")
    _close(state[1][[2, 0, 1]], torch.exp(i - m)[..., None] * k.double().view(B, H, K), 5e-6, "n")


def test_gates_of_long_and_short_portions():
    """The chain of maxima over more tokens than a block takes at a time, beside short portions."""
    from minivllm_b200.layers import mlstm as L
    H, cap, lens = 2, 9.0, [5000, 1, 2049, 4, 127]
    zs = [_gates(s, n, H, cap) for s, n in enumerate(lens)]
    b = torch.tensor([0.5, -0.25])
    m = torch.full((6, H), float("nan"), device="cuda")
    m[4] = torch.tensor([2.0, -1.0])
    chain = L.mlstm_gates(torch.cat(zs).cuda(), b.cuda(), b.cuda(), cap, _cu(lens), _i32([0, 1, 2, 3, 4]), _i32([0, 0, 0, 0, 9]), m, H)
    at = 0
    for s, (n, z) in enumerate(zip(lens, zs)):
        i = oracle.soft_cap(z[:, :H].double() + b.double(), cap)
        f = oracle.log_sigmoid(oracle.soft_cap(z[:, H:].double() + b.double(), cap))
        run, want = torch.tensor([2.0, -1.0]).double() if s == 4 else torch.zeros(H).double(), []
        for t in range(n):
            run = torch.maximum(f[t] + run, i[t])
            want.append(run)
        c = chain[at:at + n].cpu()
        assert float((c[..., 3].double() - torch.stack(want)).abs().max()) < 5e-5
        assert torch.equal(c[1:, :, 2], c[:-1, :, 3]) and torch.equal(m[s].cpu(), c[-1, :, 3])
        at += n


@pytest.mark.parametrize("chunked", [False, True], ids=["tokens", "chunks"])
def test_memory_over_many_tokens(chunked):
    """A write at the start is read out 3,000 tokens later, through many portions."""
    from minivllm_b200.layers import mlstm as L
    H, K, V, n, cap = 1, 32, 16, 3000, 15.0
    dtype = torch.bfloat16 if chunked else torch.float32
    q, k, v = (_rnd(i, n, H, D, scale=s).to(dtype) for i, (D, s) in enumerate(((K, 1.0), (K, 1e-3), (V, 1.0))))
    k[0], v[0] = _rnd(4, H, K).to(dtype), _rnd(5, H, V, scale=20.0).to(dtype)
    q = (k[:1] + 0.2 * q).to(dtype)
    z = torch.cat([torch.full((n, H), -1.0), 8.5 + 0.3 * _rnd(6, n, H)], 1)
    z[0, 0] = 6.0
    zero = torch.zeros(H, dtype=dtype)
    (o, last, _, _), = _memory_refs([(q, k, v, None, z)], H, K, V, zero, zero, cap)
    state, rows = _poison(1, H, K, V), []
    p = torch.cat([q, k, v], 2).flatten(1).cuda()
    for a in range(0, n, 500):
        at = (_cu([500]), _i32([0]), _i32([a]))
        chain = L.mlstm_gates(z[a:a + 500].cuda(), zero.cuda(), zero.cuda(), cap, *at, state[2], H)
        qs, ks, vs = p[a:a + 500].split([K, K, V], 1)
        out, den = L.mlstm_scan(qs, ks, vs, chain, *at, *state[:2], H, K, V, chunked=chunked)
        rows.append(out.double().cpu() / den.double().cpu())
    _close(torch.cat(rows)[-500:], o[-500:, 0], 6e-3 if chunked else 2e-5, "late")
    _check_state(state, last, 0, 1e-4 if chunked else 1e-5, 1e-4)


def test_padding_rows_leave_the_memory_alone():
    from minivllm_b200.layers import mlstm as L
    for H, K, V in ((2, 16, 8), (1, 9, 7)):
        state = tuple(torch.full((3, *s), 2.0, device="cuda") for s in ((H, K, V), (H, K), (H,)))
        q, k, v, g = _rnd(1, 2, 2 * H * K + 2 * H * V).cuda().split([H * K, H * K, H * V, H * V], 1)
        b = _rnd(2, H).cuda()
        out = L.mlstm_step(q, k, v, _rnd(3, 2, 11).cuda(), _rnd(5, 2 * H, 11).cuda(), b, b, 5.0, _i32([2, 1]), _i32([-1, 5]), *state, H, K, V, g, _rnd(4, H * V).cuda(), 1e-5)
        assert bool((out[0] == 0).all()) and bool((out[1] != 0).any())
        assert all(bool((t[[0, 2]] == 2.0).all()) and bool((t[1] != 2.0).any()) for t in state)


# ------------------------------------------------------------------------------------------------ norms, gates
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,vdim", [(3, 10), (4, 64), (1, 40), (12, 8), (16, 128), (2, 256), (2, 1040)])
def test_head_norm_with_denominators(heads, vdim, dtype):
    """A weight for the whole row or one that the heads share, a denominator per head, either gate."""
    from minivllm_b200.layers import group_norm as GN
    n, eps, d = 6, 1e-3, lambda t: t.double()
    y, z = _rnd(1, n, heads * vdim, dtype=dtype), _rnd(2, n, heads * vdim + 8, dtype=dtype)[:, 8:]
    den = _rnd(3, n, heads).abs() * 20 + 0.01
    for w in (_rnd(4, heads * vdim, dtype=dtype), _rnd(5, vdim, dtype=dtype)):
        full = d(w) if w.numel() == heads * vdim else d(w).repeat(heads)
        for dn in (den, None):
            r = d(y).view(n, heads, vdim) / (d(dn)[..., None] if dn is not None else 1.0)
            o = oracle.rms_norm(r, 1.0, eps).flatten(1) * full
            for act, f in (("sigmoid", oracle.sigmoid), ("silu", lambda t: t * oracle.sigmoid(t))):
                got = GN.head_norm_gate(y.cuda(), z.cuda(), w.cuda(), heads, eps, den=dn.cuda() if dn is not None else None, act=act)
                _close(got, o * f(d(z)), TOL[dtype], act)
    with pytest.raises(ValueError):
        GN.head_norm_gate(y.cuda(), z.cuda(), torch.ones(heads * vdim + 1, device="cuda", dtype=dtype), heads, eps)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_relu_gate(dtype):
    from minivllm_b200.layers import group_norm as GN
    for cols in (77, 128):
        g, u = _rnd(1, 9, cols, dtype=dtype, scale=4.0), _rnd(2, 9, cols, dtype=dtype, scale=4.0)
        _close(GN.gate_mul(u.cuda(), g.cuda(), "relu"), g.double().clamp(min=0) * u.double(), TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_relu_gate_of_grouped_products(dtype):
    """The activation is an option of the experts' products too."""
    from minivllm_b200.layers import moe
    experts, top, width, ff, n = 4, 2, 64, 40, 30
    h, w = _rnd(1, n, width, dtype=dtype), _rnd(2, experts, 2 * ff, width, dtype=dtype, scale=width ** -0.5)
    idx, _ = moe.route(_rnd(3, n, experts).cuda(), None, top)
    pos, rows, offsets = moe.sort_by_expert(idx, experts)
    x = moe.gather_rows(h.cuda(), rows)
    for tc in [False] + ([True] if dtype == torch.bfloat16 else []):
        got = moe.grouped_linear(x, w.cuda(), offsets, gated=True, tensor_cores=tc, act="relu").cpu()
        want = torch.zeros(n * top, ff, dtype=torch.float64)
        for t in range(n):
            for k in range(top):
                z = w[int(idx[t, k])].double() @ h[t].double()
                want[int(pos[t, k])] = z[:ff].clamp(min=0) * z[ff:]
        _close(got, want, 1e-5 if dtype == torch.float32 else 1.6e-2)
