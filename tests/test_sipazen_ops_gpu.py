"""Every mechanism of the Sipazen family alone, on the GPU, against the plain oracle's function for it."""
import math

import pytest
import torch

from oracle import sipazen_oracle as oracle

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


# ------------------------------------------------------------------------------------------------ norms and gates
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width,groups", [(90, 3), (64, 1), (2048, 4), (96, 12), (1536, 3), (8192, 2), (40, 5), (768, 8)])
def test_residual_norms(width, groups, dtype):
    """Both forms of the step between sublayers and the first norm, on rows in registers and in shared memory, chunked
    and element by element."""
    from minivllm_b200.layers import group_norm as GN
    rows, eps, mult = 7, 1e-4, 0.37
    y, gate, b = _rnd(1, rows, width, dtype=dtype), _rnd(2, rows, width, dtype=dtype), _rnd(3, width, dtype=dtype)
    w1, w2, x = _rnd(4, width, dtype=dtype), _rnd(5, width, dtype=dtype), _rnd(6, rows, width)
    d = lambda t: t.double()
    for use_gate in (True, False):
        v = d(y) * oracle.sigmoid(d(gate) + d(b)) if use_gate else d(y)
        want_x = d(x) + mult * oracle.grouped_rms_norm(v, d(w1), groups, eps)
        gx = x.cuda()
        h = GN.gated_residual_norm(gx, y.cuda(), gate.cuda() if use_gate else None, b.cuda(), w1.cuda(), w2.cuda(), mult, groups, eps)
        _close(gx, want_x, TOL[torch.float32] * (10 if dtype == torch.bfloat16 else 1), "residual")
        _close(h, oracle.grouped_rms_norm(want_x, d(w2), groups, eps), TOL[dtype], "next input")
    table, ids = _rnd(7, 11, width, dtype=dtype), torch.tensor([3, 0, 10, 3, 7, 1, 2])
    gx, h = GN.embed_norm(ids.cuda(), table.cuda(), w2.cuda(), groups, eps)
    assert torch.equal(gx.cpu(), table[ids].float())
    _close(h, oracle.grouped_rms_norm(d(table[ids]), d(w2), groups, eps), TOL[dtype], "embedding")
    top = 3
    pos = torch.randperm(rows * top, generator=torch.Generator().manual_seed(8)).to(torch.int32).view(rows, top)
    er, tw = _rnd(9, rows * top, width, dtype=dtype), _rnd(10, rows, top).abs()
    sh, sg = _rnd(11, rows, width, dtype=dtype), _rnd(12, rows, 1, dtype=dtype)
    v = (d(tw)[..., None] * d(er)[pos.long()]).sum(1) + oracle.sigmoid(d(sg)) * d(sh)
    want_x = d(x) + mult * oracle.grouped_rms_norm(v * oracle.sigmoid(d(gate) + d(b)), d(w1), groups, eps)
    gx = x.cuda()
    h = GN.moe_residual_norm(gx, er.cuda(), pos.cuda(), tw.cuda(), sh.cuda(), sg.cuda(), gate.cuda(), b.cuda(), w1.cuda(), w2.cuda(),
                             mult, groups, eps)
    _close(gx, want_x, TOL[torch.float32] * (10 if dtype == torch.bfloat16 else 1), "residual, experts")
    _close(h, oracle.grouped_rms_norm(want_x, d(w2), groups, eps), TOL[dtype], "next input, experts")
    _close(GN.gated_group_norm(y.cuda(), gate.cuda(), w1.cuda(), groups, eps),
           oracle.grouped_rms_norm(d(y) * oracle.silu(d(gate)), d(w1), groups, eps), TOL[dtype], "gated norm")
    _close(GN.gate_mul(y.cuda(), gate.cuda()), d(y) * oracle.sigmoid(d(gate)), TOL[dtype], "sigmoid gate")
    _close(GN.gate_mul(y.cuda(), gate.cuda(), "silu"), d(y) * oracle.silu(d(gate)), TOL[dtype], "silu gate")


# ------------------------------------------------------------------------------------------------ latent rows
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,dim,rot,rope,rank", [(3, 10, 6, 6, 14), (4, 16, 16, 16, 64), (2, 8, 32, 32, 40), (2, 12, 16, 8, 24),
                                                     (5, 128, 64, 64, 512), (1, 24, 48, 48, 1000)])
def test_latent_preparation(heads, dim, rot, rope, rank, dtype):
    from minivllm_b200.layers import latent_attention as LA
    pos = torch.tensor([0, 1, 17, 400, 5000])
    n, eps, base = len(pos), 1e-3, 700.0
    q, down, w = _rnd(1, n, heads * (dim + rot), dtype=dtype), _rnd(2, n, rank + rot, dtype=dtype), _rnd(3, rank, dtype=dtype)
    slots = torch.tensor([9, -1, 0, 31, 12])
    cache = torch.full((4, 8, rank + rot), 7.0, dtype=dtype, device="cuda")
    ct, st = LA.rope_table(base, rope, 5001, torch.device("cuda"))
    gq = q.cuda()
    lat = LA.latent_prep(gq, down.cuda(), w.cuda(), pos.cuda(), ct, st, heads, dim, rot, rope, rank, eps, cache, slots.cuda())
    want_q, want = q.double().view(n, heads, dim + rot).clone(), torch.zeros(n, rank + rot, dtype=torch.float64)
    want[:, :rank] = oracle.grouped_rms_norm(down[:, :rank].double(), w.double(), 1, eps)
    for i, p in enumerate(pos.tolist()):
        want[i, rank:] = oracle.rotate(down[i, rank:].double(), p, base, rope)
        want_q[i, :, dim:] = oracle.rotate(want_q[i, :, dim:], p, base, rope)
    tol = 2e-6 if dtype == torch.float32 else 6e-3
    _close(lat, want, tol, "latent rows")
    _close(gq.view(n, heads, dim + rot), want_q, tol, "queries")
    flat = cache.view(32, -1)
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(flat[s], lat[i])
    untouched = [s for s in range(32) if s not in slots.tolist()]
    assert bool((flat[untouched] == 7.0).all())


def _paged(rows_per_seq, bs, row, dtype, seed=0, spare=3):
    """Latent rows of several sequences in a paged cache with shuffled blocks: cache, tables, rows by sequence."""
    g = torch.Generator().manual_seed(seed)
    need = [-(-n // bs) for n in rows_per_seq]
    perm = torch.randperm(sum(need) + spare, generator=g).tolist()
    cache = torch.zeros(sum(need) + spare, bs, row, dtype=dtype)
    tables = torch.full((len(need), max(need)), -1, dtype=torch.int32)
    data = []
    for s, n in enumerate(rows_per_seq):
        lat = torch.randn(n, row, generator=g).to(dtype)
        data.append(lat)
        for b in range(need[s]):
            blk = perm.pop()
            tables[s, b] = blk
            part = lat[b * bs:(b + 1) * bs]
            cache[blk, :len(part)] = part
    return cache.cuda(), tables.cuda(), data


def _attend(ql, qr, lat, rank, scale, sink, visible):
    """Absorbed attention of one row: ql (heads, rank), qr (heads, rot) on the first `visible` rows."""
    k = lat[:visible].double()
    s = (torch.cat([ql, qr], -1).double() @ k.T) * scale
    top = torch.maximum(s.max(-1).values, sink.double())[:, None]
    e = torch.exp(s - top)
    return (e / (e.sum(-1, keepdim=True) + torch.exp(sink.double()[:, None] - top))) @ k[:, :rank]


def _standout(q_row, lat, key, gain):
    """Makes one key answer one query row far above all others."""
    lat[key] = (q_row.float() / q_row.float().norm() * gain).to(lat.dtype)


@pytest.mark.parametrize("heads,rank,rot,bs", [(16, 512, 64, 64), (5, 64, 32, 16), (20, 256, 64, 32), (3, 112, 16, 8), (33, 128, 0, 128),
                                               (16, 512, 64, 256)])
def test_latent_decode(heads, rank, rot, bs):
    """Unequal sequences (from one key to thousands, cut between workers), a padding row, a key that stands out at the
    start, at every kind of border and at the end of a sequence, sinks of any size."""
    from minivllm_b200.layers import latent_attention as LA
    bf = torch.bfloat16
    lens = [1, 31, 32, 33, 2 * bs, 2 * bs + 1, 700, 3000, 129, 5]
    cache, tables, data = _paged(lens, bs, rank + rot, bf)
    n, scale = len(lens), (rank + rot) ** -0.5
    ql, qr = _rnd(1, n + 1, heads, rank, dtype=bf), _rnd(2, n + 1, heads, max(rot, 1), dtype=bf)[:, :, :rot]
    sink = _rnd(3, heads, dtype=bf, scale=3.0)
    for s, key in ((6, 0), (7, 2048), (7, 2999), (5, 2 * bs), (4, bs - 1), (8, 128)):
        q = torch.cat([ql[s, 0], qr[s, 0]])
        lat = data[s]
        _standout(q, lat, key, 40.0)
        cache[tables[s, key // bs].long(), key % bs] = lat[key].cuda()
    tables = torch.cat([tables, torch.full_like(tables[:1], -1)])     # a padding row: no block, position 0
    pos = torch.tensor([l - 1 for l in lens] + [0])
    got = LA.latent_decode(ql.cuda(), qr.cuda(), cache, tables, pos.cuda(), sink.cuda(), scale)
    assert got is not None
    rows = LA.latent_attention_rows(ql.cuda(), qr.cuda(), cache, tables, None, pos.cuda(), sink.cuda(), scale)
    for s in range(n):
        want = _attend(ql[s], qr[s], data[s], rank, scale, sink, lens[s])
        _close(got[s], want, 1e-2, f"sequence {s}")
        _close(rows[s], want, 1e-2, f"sequence {s}, general kernel")
    assert float(got[n].abs().max()) == 0.0
    alone = LA.latent_decode(ql[7:8].cuda(), qr[7:8].cuda(), cache, tables[7:8], pos[7:8].cuda(), sink.cuda(), scale)
    _close(alone[0], got[7].double().cpu(), 1e-2, "alone")
    no_sink = LA.latent_decode(ql[:n].cuda(), qr[:n].cuda(), cache, tables[:n], pos[:n].cuda(), None, scale)
    _close(no_sink[0], data[0][0, :rank].double().expand(heads, rank), 1e-2, "one key, no sink")


@pytest.mark.parametrize("heads,dim,rot,vdim", [(2, 128, 64, 128), (3, 64, 64, 64), (2, 40, 24, 72), (1, 16, 8, 8), (2, 64, 0, 128),
                                                (2, 192, 0, 56)])
def test_latent_prefill(heads, dim, rot, vdim):
    """Packed prompts and portions behind cached tokens; lengths around the tile borders; one key that stands out for
    the last query, the diagonal, and the key just behind a query, which must not be seen."""
    from minivllm_b200.layers import latent_attention as LA
    bf = torch.bfloat16
    q_lens = [1, 127, 128, 129, 257, 2, 300, 40]
    past = [0, 0, 0, 200, 0, 255, 77, 1000]
    k_lens = [a + b for a, b in zip(q_lens, past)]
    T, K, scale = sum(q_lens), sum(k_lens), 1.3 * (dim + rot) ** -0.5
    q, kv, kr = _rnd(1, T, heads * (dim + rot), dtype=bf), _rnd(2, K, heads * (dim + vdim), dtype=bf), _rnd(3, K, max(rot, 8), dtype=bf)
    kr = kr[:, :rot]
    sink = _rnd(4, heads, dtype=bf, scale=2.0)
    cuq, cuk = _cu(q_lens), _cu(k_lens)
    qo = kv_o = 0
    for n, p in zip(q_lens, past):          # key 0, the query's own key and the next one, for the last and a middle query
        for i in {n - 1, n // 2}:
            for j, gain in ((0, 9.0), (p + i, 6.0), (min(p + i + 1, p + n - 1), 30.0)):
                row = q[qo + i, :dim].float()
                kv[kv_o + j, :dim] = (row / row.norm() * gain).to(bf)
        qo, kv_o = qo + n, kv_o + n + p
    pad = torch.zeros(K, rot + 8, dtype=bf, device="cuda")
    pad[:, 8:] = kr.cuda()
    got = LA.latent_prefill(q.cuda(), kv.cuda(), pad[:, 8:] if rot else pad, cuq, cuk, heads, dim, rot, vdim, scale, sink.cuda())
    qo = kv_o = 0
    for n, p in zip(q_lens, past):
        qs = q[qo:qo + n].double().view(n, heads, dim + rot)
        ks = kv[kv_o:kv_o + n + p, :heads * dim].double().view(-1, heads, dim)
        vs = kv[kv_o:kv_o + n + p, heads * dim:].double().view(-1, heads, vdim)
        krs = kr[kv_o:kv_o + n + p].double()
        for h in range(heads):
            s = (qs[:, h, :dim] @ ks[:, h].T + qs[:, h, dim:] @ krs.T) * scale
            s = s.masked_fill(torch.arange(n + p)[None, :] > (torch.arange(n) + p)[:, None], -math.inf)
            top = torch.maximum(s.max(-1, keepdim=True).values, sink[h].double())
            e = torch.exp(s - top)
            want = (e / (e.sum(-1, keepdim=True) + torch.exp(sink[h].double() - top))) @ vs[:, h]
            _close(got[qo:qo + n].view(n, heads, vdim)[:, h], want, 1.2e-2, f"{n} queries behind {p}, head {h}")
        qo, kv_o = qo + n, kv_o + n + p


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_general_latent_attention_and_gather(dtype):
    """The kernel for any sizes: several query rows per sequence behind cached tokens, a rank beyond 512, and the packed
    gather of cached rows."""
    from minivllm_b200.layers import latent_attention as LA
    heads, rank, rot, bs = 5, 520, 24, 8
    k_lens, q_lens = [40, 3, 129], [5, 3, 65]
    cache, tables, data = _paged(k_lens, bs, rank + rot, dtype)
    T, scale = sum(q_lens), 0.05
    ql, qr, sink = _rnd(1, T, heads, rank, dtype=dtype), _rnd(2, T, heads, rot, dtype=dtype), _rnd(3, heads, dtype=dtype)
    pos = torch.cat([torch.arange(k - n, k) for k, n in zip(k_lens, q_lens)])
    got = LA.latent_attention_rows(ql.cuda(), qr.cuda(), cache, tables, _cu(q_lens), pos.cuda(), sink.cuda(), scale)
    at = 0
    for s, n in enumerate(q_lens):
        for i in range(n):
            want = _attend(ql[at], qr[at], data[s], rank, scale, sink, int(pos[at]) + 1)
            _close(got[at], want, 4e-6 if dtype == torch.float32 else 1e-2, f"sequence {s} row {i}")
            at += 1
    packed = LA.latent_gather(cache, _cu(k_lens), sum(k_lens), tables)
    assert torch.equal(packed.cpu(), torch.cat(data))


# ------------------------------------------------------------------------------------------------ state space
def _ssm_inputs(lens, heads, P, N, G, taps, dtype, seed=0, slow=False):
    T, ch = sum(lens), heads * P + 2 * G * N
    u, dt = _rnd(seed, T, ch, dtype=dtype), _rnd(seed + 1, T, heads, dtype=dtype)
    cw, cb = _rnd(seed + 2, ch, taps, dtype=dtype, scale=taps ** -0.5), _rnd(seed + 3, ch, dtype=dtype, scale=0.2)
    A = (_rnd(seed + 4, heads) - (9.0 if slow else 1.0)).to(dtype)
    db, D = (_rnd(seed + 5, heads) - 1.0).to(dtype), _rnd(seed + 6, heads, dtype=dtype)
    return u, dt, cw, cb, A, db, D


def _ssm_oracle(u, dt, cw, cb, A, db, D, heads, P, N, G, round_conv=None):
    d = lambda t: t.double()
    L = u.shape[0]
    xbc = oracle.causal_conv_silu(d(u), d(cw), d(cb))
    if round_conv is not None:
        xbc = xbc.to(round_conv).double()
    x = xbc[:, :heads * P].reshape(L, heads, P)
    B, C = xbc[:, heads * P:heads * P + G * N].reshape(L, G, N), xbc[:, heads * P + G * N:].reshape(L, G, N)
    y, S = oracle.ssm_scan(x, B, C, oracle.softplus(d(dt) + d(db)), d(A), d(D))
    return y.reshape(L, heads * P), S


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,P,N,G,taps", [(4, 64, 128, 2, 4), (3, 24, 32, 1, 2), (6, 40, 64, 3, 3), (2, 12, 20, 1, 4), (2, 10, 14, 2, 5),
                                              (1, 72, 128, 1, 1)])
@pytest.mark.parametrize("slow", [False, True], ids=["fast", "slow"])
def test_state_space_portions_and_steps(heads, P, N, G, taps, dtype, slow):
    """Portions cut at and around the chunk length with the state carried in slots, several sequences at once, and
    single steps; `slow` decays keep the first token alive to the end of the sequence."""
    from minivllm_b200.layers import mamba2 as M
    lens = [150, 67, 3]
    seqs = [_ssm_inputs([n], heads, P, N, G, taps, dtype, seed=10 * i, slow=slow) for i, n in enumerate(lens)]
    shared = seqs[0][2:]
    want = [_ssm_oracle(s[0], s[1], *shared, heads, P, N, G, dtype if dtype == torch.bfloat16 else None) for s in seqs]
    cw, cb, A, db, D = (t.cuda() for t in shared)
    ch = heads * P + 2 * G * N
    conv = torch.full((5, max(taps - 1, 1), ch), 50.0, dtype=dtype, device="cuda")[:, :taps - 1]
    conv = conv.contiguous()
    ssm = torch.full((5, heads, N, P), 50.0, device="cuda")             # stale contents of the slots
    slot_of, at, out = [3, 0, 4], [0, 0, 0], [[], [], []]
    can_step = P % 4 == 0 and N % 4 == 0
    plan = [{0: 64, 1: 2}, {0: 1}, {0: 63, 2: 2}, {1: 64}, {0: 2, 1: 1, 2: 1}, {0: 20}]
    for step in plan:
        ids = sorted(step, key=lambda i: step[i] != 1)                  # one-token sequences first, as in the engine
        n1 = sum(step[i] == 1 for i in ids)
        u = torch.cat([seqs[i][0][at[i]:at[i] + step[i]] for i in ids]).cuda()
        dt = torch.cat([seqs[i][1][at[i]:at[i] + step[i]] for i in ids]).cuda()
        slots = torch.tensor([slot_of[i] for i in ids], dtype=torch.int32, device="cuda")
        starts = torch.tensor([at[i] for i in ids], dtype=torch.int32, device="cuda")
        cu = _cu([step[i] for i in ids])
        y = torch.zeros(u.shape[0], heads * P, dtype=dtype, device="cuda")
        dims = (heads, P, N, G)
        if n1 and can_step:
            M.ssm_step(u[:n1], cw, cb, conv, dt[:n1], db, A, D, slots[:n1], starts[:n1], ssm, *dims, out=y[:n1])
        elif n1:
            xbc = M.conv_silu(u[:n1], cw, cb, None, slots[:n1], starts[:n1], conv)
            M.ssm_scan(xbc, dt[:n1], db, A, D, None, slots[:n1], starts[:n1], ssm, *dims, out=y[:n1])
        if len(ids) > n1:
            c = (cu[n1:] - cu[n1]).contiguous()
            xbc = M.conv_silu(u[n1:], cw, cb, c, slots[n1:], starts[n1:], conv)
            M.ssm_scan(xbc, dt[n1:], db, A, D, c, slots[n1:], starts[n1:], ssm, *dims, out=y[n1:])
        if taps > 1:
            M.conv_state_update(conv, u, taps, cu, slots, starts)
        o = 0
        for i in ids:
            out[i].append(y[o:o + step[i]].cpu())
            o, at[i] = o + step[i], at[i] + step[i]
    tol = 5e-6 if dtype == torch.float32 else 1.5e-2
    for i, n in enumerate(lens):
        assert at[i] == n
        _close(torch.cat(out[i]), want[i][0], tol, f"sequence {i}")
        # the convolution's rounding to bf16 differs where its fp32 and fp64 results straddle a rounding border
        _close(ssm[slot_of[i]], want[i][1], 5e-6 if dtype == torch.float32 else 4e-3, f"state {i}")
    assert float(ssm[1].min()) == 50.0 and float(ssm[2].min()) == 50.0


def test_state_is_not_rounded_to_bf16():
    """A state that grows by small steps: with bf16 anywhere in the recurrence the steps would be lost or biased."""
    from minivllm_b200.layers import mamba2 as M
    heads, P, N, G, L = 2, 64, 64, 1, 640
    bf = torch.bfloat16
    xbc = torch.cat([torch.full((L, heads * P), 0.00390625), torch.full((L, 2 * N), 1.0)], 1).to(bf).cuda()
    dt, db = torch.full((L, heads), -3.0, dtype=bf, device="cuda"), torch.zeros(heads, dtype=bf, device="cuda")
    A, D = torch.full((heads,), -20.0, dtype=bf, device="cuda"), torch.zeros(heads, dtype=bf, device="cuda")
    one = torch.zeros(1, dtype=torch.int32, device="cuda")
    want = L * float(oracle.softplus(torch.tensor(-3.0, dtype=torch.float64))) * 0.00390625
    for chunked in (True, False):
        ssm = torch.zeros(1, heads, N, P, device="cuda")
        M.ssm_scan(xbc, dt, db, A, D, _cu([L]), one, one, ssm, heads, P, N, G, chunked=chunked)
        assert float((ssm / want - 1).abs().max()) < 2e-5, chunked


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("experts,top", [(5, 3), (7, 1), (64, 6), (130, 8), (600, 2), (4, 4)])
def test_router(experts, top):
    from minivllm_b200.layers import moe
    h, W, b = _rnd(1, 300, 48), _rnd(2, experts, 48), _rnd(3, experts)
    z = (h.double() @ W.double().T).float()
    idx, weight = moe.route(z.cuda(), b.cuda(), top)
    want_i, want_w = oracle.route(z.double(), torch.eye(experts, dtype=torch.float64), b.double(), top)
    assert torch.equal(idx.cpu().long(), want_i)
    _close(weight, want_w, 1e-5, "weights")
    tie = torch.zeros(3, experts, device="cuda")
    idx, weight = moe.route(tie, None, top)
    assert idx.tolist() == [list(range(top))] * 3 and float((weight - 1 / top).abs().max()) < 1e-6


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("experts,top,tokens,width,ff", [(5, 3, 40, 48, 22), (8, 2, 700, 192, 136), (64, 6, 9, 128, 64), (3, 2, 1500, 72, 264),
                                                        (16, 4, 3, 64, 8), (4, 1, 130, 200, 128)])
def test_experts(experts, top, tokens, width, ff, dtype):
    """Sort, gather and both grouped products; experts without tokens, with one, and with several tiles."""
    from minivllm_b200.layers import moe
    h = _rnd(1, tokens, width, dtype=dtype)
    gate_up, down = _rnd(2, experts, 2 * ff, width, dtype=dtype, scale=width ** -0.5), _rnd(3, experts, width, ff, dtype=dtype, scale=ff ** -0.5)
    z = _rnd(4, tokens, experts)
    z[:, 0] -= 100.0                                   # nobody chooses expert 0
    if top < experts - 1:
        z[:, 1] -= 50.0
        z[0, 1] += 200.0                               # one token chooses expert 1
    idx, weight = moe.route(z.cuda(), None, top)
    pos, row_token, offsets = moe.sort_by_expert(idx, experts)
    e, p = idx.cpu().long(), pos.cpu().long()
    counts = torch.bincount(e.view(-1), minlength=experts)
    assert offsets.tolist() == [0] + counts.cumsum(0).tolist()
    assert sorted(p.view(-1).tolist()) == list(range(tokens * top))
    order = torch.empty(tokens * top, dtype=torch.long)
    order[p.view(-1)] = torch.arange(tokens * top)
    assert torch.equal(row_token.cpu().long(), order // top)
    assert torch.equal(order, torch.argsort(e.view(-1), stable=True))
    x = moe.gather_rows(h.cuda(), row_token)
    assert torch.equal(x.cpu(), h[row_token.cpu().long()])
    forms = [False] + ([True] if dtype == torch.bfloat16 and width % 8 == 0 and ff % 8 == 0 else [])
    row_e = e.view(-1)[order]
    hx = h[row_token.cpu().long()].double()
    for tc in forms:
        act = moe.grouped_linear(x, gate_up.cuda(), offsets, gated=True, tensor_cores=tc)
        out = moe.grouped_linear(act, down.cuda(), offsets, tensor_cores=tc)
        for k in range(experts):
            rows = row_e == k
            if not rows.any():
                continue
            g, u = hx[rows] @ gate_up[k, :ff].double().T, hx[rows] @ gate_up[k, ff:].double().T
            _close(act[rows.cuda()], oracle.silu(g) * u, 3e-6 if dtype == torch.float32 else 8e-3, f"gated product of expert {k}")
            _close(out[rows.cuda()], act[rows.cuda()].double().cpu() @ down[k].double().T, 3e-6 if dtype == torch.float32 else 8e-3,
                   f"product of expert {k}")


# ------------------------------------------------------------------------------------------------ sampling in 32-bit
def test_fp32_greedy_and_sampled_rows():
    from minivllm_b200.layers import sampler
    z = _rnd(1, 6, 1003).cuda()
    assert torch.equal(sampler.greedy_tokens(z), z.argmax(-1))
    step = torch.zeros(1, dtype=torch.int64, device="cuda")
    t = torch.tensor([0.0, 0.0, 1.0, 1.0, 0.5, 2.0], device="cuda")
    got = sampler.sampled_tokens(z, t, 7, step)
    assert torch.equal(got[:2], z[:2].argmax(-1)) and bool(((got >= 0) & (got < 1003)).all())
    assert torch.equal(got, sampler.sampled_tokens(z, t, 7, step))
