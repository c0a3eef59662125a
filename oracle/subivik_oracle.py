"""Plain restatement of the Subivik decoder on the CPU: one function per mechanism, written for reading, not for speed, and
sharing no code with the package.  A whole sequence goes in, position by position where the mechanism is recurrent; there is
no cache, no batching and no cutting into portions.

Notation: a sequence is an (L, width) matrix, weights are (out, in) and applied as `x @ W.T`.  `w` is a dict of tensors
under the checkpoint's names; everything is computed in the dtype of those tensors (float64 by default).
"""
import math

import torch


def sigmoid(z):
    return torch.exp(-torch.logaddexp(torch.zeros_like(z), -z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.logaddexp(torch.zeros_like(z), z)


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def dynamic_tanh(x, alpha, weight, bias):
    return torch.tanh(alpha * x) * weight + bias


def position_vectors(L, width, dtype):
    out = torch.zeros(L, width, dtype=torch.float64)
    for p in range(L):
        for c in range(width):
            angle = p * 10000.0 ** (-2 * (c // 2) / width)
            out[p, c] = math.cos(angle) if c % 2 else math.sin(angle)
    return out.to(dtype)


# ---------------------------------------------------------------------------------------------- capped attention, mixed heads
def capped_weights(q, k, r1, r2, scale, cap):
    """q (L, H, d), k (L, G, d) -> weights (H, L, L): causal softmax of capped scores minus a bias that grows with the
    logarithm of the distance."""
    L, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(H, L, L, dtype=q.dtype)
    for head in range(H):
        for i in range(L):
            s = (k[:i + 1, head // (H // G)] @ q[i, head]) * scale
            s = cap * torch.tanh(s / cap)
            distance = (i - torch.arange(i + 1)).to(q.dtype)
            s = s - r1[head] * torch.log(1.0 + r2[head] * distance)
            e = torch.exp(s - s.max())
            out[head, i, :i + 1] = e / e.sum()
    return out


def mix_heads(weights, talk):
    """weights (H, L, L): every head takes a combination of all heads' weights."""
    return torch.einsum("hg,gij->hij", talk, weights)


def capped_attention(h, w, p, m):
    L, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(L, H, d)
    k = (h @ w[p + "k"].T).reshape(L, G, d)
    v = (h @ w[p + "v"].T).reshape(L, G, vd)
    a = mix_heads(capped_weights(q, k, w[p + "r1"], w[p + "r2"], m["scale"], m["softcap"]), w[p + "talk"])
    o = torch.stack([a[head] @ v[:, head // (H // G)] for head in range(H)], dim=1)
    return o.reshape(L, H * vd) @ w[p + "o"].T


# ---------------------------------------------------------------------------------------------- time mixing
def shift_mix(h, mu):
    """Every token moves towards the token before it (zeros before the first), channel by channel."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def bonus_scan(r, k, v, decay, u):
    """r, k, decay (L, H, K), v (L, H, V), u (H, K): a token's read-out sees the state before it and, weighted by u, its own
    entry.  Returns the read-outs (L, H, V) and the last state (H, K, V)."""
    L, H, K = r.shape
    S = torch.zeros(H, K, v.shape[2], dtype=r.dtype)
    out = torch.zeros_like(v)
    for t in range(L):
        entry = k[t][:, :, None] * v[t][:, None, :]
        out[t] = (r[t][:, :, None] * (S + u[:, :, None] * entry)).sum(1)
        S = decay[t][:, :, None] * S + entry
    return out, S


def time_mixing(h, w, p, m, eps):
    L, H, K = h.shape[0], m["heads"], m["dim"]
    x = {n: shift_mix(h, w[p + "mu." + n]) for n in "rkvgw"}
    r, k, v = ((x[n] @ w[p + n].T).reshape(L, H, K) for n in "rkv")
    z = torch.tanh(x["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    o, _ = bonus_scan(r, k, v, torch.exp(-torch.exp(z)).reshape(L, H, K), w[p + "u"])
    o = rms_norm(o, 1.0, eps).reshape(L, H * K) * w[p + "norm"]
    return (o * silu(x["g"] @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return m["left_scale"] * capped_attention(h, w, p + "left.", m["left"]) + \
        m["right_scale"] * time_mixing(h, w, p + "right.", m["right"], eps)


# ---------------------------------------------------------------------------------------------- differential attention
def chunk_attention(q, k, v, scale, size):
    """One map: q (L, H, d), k (L, G, d), v (L, G, vd) -> (L, H, vd); a position sees its own chunk up to itself."""
    L, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for i in range(L):
        j0 = i // size * size
        for head in range(H):
            g = head // (H // G)
            s = (k[j0:i + 1, g] @ q[i, head]) * scale
            e = torch.exp(s - s.max())
            out[i, head] = (e / e.sum()) @ v[j0:i + 1, g]
    return out


def difference_factor(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def keys_values(h, w, p, m, eps):
    """Normed keys (L, G, 2, dim) and values (L, G, vdim), as a later layer may use them too."""
    L, G, d, vd = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    k = rms_norm((h @ w[p + "k"].T).reshape(L, G, 2, d), w[p + "k.norm"], eps)
    return k, (h @ w[p + "v"].T).reshape(L, G, vd)


def differential_attention(h, w, p, m, eps, kv=None):
    """Returns the result and the keys and values used (`kv`: those of an earlier layer)."""
    L, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    k, v = kv if kv is not None else keys_values(h, w, p, m, eps)
    q = rms_norm((h @ w[p + "q"].T).reshape(L, H, 2, d), w[p + "q.norm"], eps)
    a1, a2 = (chunk_attention(q[:, :, n], k[:, :, n], v, m["scale"], m["mask"]["size"]) for n in (0, 1))
    lam = difference_factor(*(w[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
    o = rms_norm(a1 - lam * a2, 1.0, eps) * (1.0 - m["diff"])
    return (o.reshape(L, H * vd) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T, (k, v)


# ---------------------------------------------------------------------------------------------- feed-forward
def xielu(z, p, q):
    up = softplus(p) * z * z + 0.5 * z
    down = (0.5 + softplus(q)) * (torch.expm1(z) - z) + 0.5 * z
    return torch.where(z > 0, up, down)


def dense(h, w, p, spec):
    return xielu(h @ w[p + "up"].T, w[p + "act"][0], w[p + "act"][1]) @ w[p + "down"].T


def route(z, top, scale):
    """Chosen experts (L, top), best first, and their weights: probabilities over all experts times `scale`."""
    s = torch.softmax(z, dim=-1)
    idx = s.argsort(dim=-1, descending=True, stable=True)[:, :top]
    return idx, s.gather(1, idx) * scale


def moe(h, w, p, spec):
    r = spec["router"]
    idx, weight = route(h @ w[p + "router"].T, r["top"], r["scale"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for n in range(idx.shape[1]):
            e = f"{p}e{int(idx[t, n])}."
            out[t] += weight[t, n] * ((silu(h[t] @ w[e + "gate"].T) * (h[t] @ w[e + "up"].T)) @ w[e + "down"].T)
    return out


# ---------------------------------------------------------------------------------------------- model
def forward(config, weights, token_ids, dtype=torch.float64, per_layer=None):
    """Logits (L, vocab).  `per_layer`, a list, receives the residual stream after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    norm = lambda x, name: dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])
    x = w["embed"][torch.as_tensor(token_ids)]
    x = x + position_vectors(x.shape[0], x.shape[1], dtype)
    kept, feed_forwards = {}, {"dense": dense, "moe": moe}
    for i, layer in enumerate(config["layers"]):
        l, m = f"l{i}.", layer["mixer"]
        h = norm(x, l + "norm1")
        if layer["type"] == "parallel":
            y = parallel(h, w, l + "mix.", m, eps)
        else:
            y, kept[i] = differential_attention(h, w, l + "mix.", m, eps, kept[m["kv_from"]] if "kv_from" in m else None)
        x = x + y
        if layer.get("mlp"):
            x = x + feed_forwards[layer["mlp"]["kind"]](norm(x, l + "norm2"), w, l + "mlp.", layer["mlp"])
        if per_layer is not None:
            per_layer.append(x)
    return norm(x, "final.norm") @ w["embed"].T


def random_weights(config, seed=0, rank=5):
    """Checkpoint tensors of a configuration from a seed, bfloat16, with every mechanism visible in the output (scores that
    the cap bends, biases of the scores' size, heads that mix strongly, decays between slow and fast, router logits far
    apart)."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (gain / math.sqrt(i))

    def around(n, mean, spread):
        return mean + spread * torch.randn(n, generator=g)

    W = config["width"]
    w = {"embed": torch.randn(config["vocab"], W, generator=g)}

    def norm(name):
        w[name], w[name + ".b"] = around(W, 1.0, 0.2), around(W, 0.0, 0.2)
        w[name + ".alpha"] = around(1, 0.7, 0.2)[0]

    norm("final.norm")
    for i, layer in enumerate(config["layers"]):
        l, m = f"l{i}.", layer["mixer"]
        p = l + "mix."
        norm(l + "norm1")
        if layer["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, d, vd = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "left."
            w.update({q + "q": mat(H * d, W, 3.0), q + "k": mat(G * d, W, 3.0), q + "v": mat(G * vd, W, 1.5),
                      q + "r1": torch.rand(H, generator=g) * 1.2, q + "r2": torch.rand(H, generator=g) + 0.1,
                      q + "talk": torch.eye(H) + mat(H, H, 0.8), q + "o": mat(W, H * vd)})
            H, K = b["heads"], b["dim"]
            q = p + "right."
            for n in "rkvgw":
                w[q + "mu." + n] = torch.rand(W, generator=g)
            for n in "rkvg":
                w[q + n] = mat(H * K, W)
            w.update({q + "w1": mat(rank, W), q + "w2": mat(H * K, rank), q + "w0": around(H * K, -2.0, 2.0),
                      q + "u": around(H * K, 0.5, 0.5).reshape(H, K), q + "norm": around(H * K, 1.0, 0.1), q + "o": mat(W, H * K)})
        else:
            H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w.update({p + "q": mat(H * 2 * d, W), p + "q.norm": around(d, 1.5, 0.3), p + "g": mat(H * vd, W), p + "o": mat(W, H * vd)})
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[p + n] = around(d, 0.0, 0.1)
            if "kv_from" not in m:
                w.update({p + "k": mat(G * 2 * d, W), p + "k.norm": around(d, 1.5, 0.3), p + "v": mat(G * vd, W)})
        e = layer.get("mlp")
        if not e:
            continue
        norm(l + "norm2")
        p = l + "mlp."
        if e["kind"] == "dense":
            w.update({p + "up": mat(e["ff"], W), p + "down": mat(W, e["ff"]), p + "act": around(2, 0.3, 0.5)})
        else:
            w[p + "router"] = mat(e["router"]["experts"], W, 3.0)
            ff = e["expert"]["ff"]
            for n in range(e["router"]["experts"]):
                w.update({f"{p}e{n}.gate": mat(ff, W, 1.5), f"{p}e{n}.up": mat(ff, W, 1.5), f"{p}e{n}.down": mat(W, ff)})
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
