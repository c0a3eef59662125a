"""Plain restatement of the Fozerax decoder on the CPU: one function per mechanism, written for reading, not for speed,
and sharing no code with the package.  A whole sequence goes in, position by position where the mechanism is recurrent;
there is no cache, no batching and no cutting into portions.

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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


# ---------------------------------------------------------------------------------------------- gated linear attention
def channel_decay(z, tau):
    return sigmoid(z) ** (1.0 / tau)


def gla_scan(q, k, v, alpha):
    """q, k, alpha (L, heads, K), v (L, heads, V) -> read-outs (L, heads, V) and the last state (heads, K, V)."""
    L, H, K = q.shape
    S = torch.zeros(H, K, v.shape[2], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(L):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (q[t][:, :, None] * S).sum(1)
    return out, S


def gla(h, w, p, m, eps):
    L, H, K, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(L, H, K) * K ** -0.5
    k = (h @ w[p + "k"].T).reshape(L, H, K)
    v = (h @ w[p + "v"].T).reshape(L, H, V)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    o, _ = gla_scan(q, k, v, channel_decay(z, m["tau"]).reshape(L, H, K))
    o = rms_norm(o, w[p + "norm"], eps).reshape(L, H * V)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---------------------------------------------------------------------------------------------- windowed attention
def distance_bucket(n, buckets, bias_max):
    """The first half of the buckets holds one distance each, the rest grow geometrically up to bias_max."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(bias_max / half) * (buckets - half)))


def windowed_attention(q, k, v, rel, sink, scale, window, bias_max):
    """q (L, H, d), k (L, G, d), v (L, G, vd), rel (buckets, H), sink (H,) -> (L, H, vd)."""
    L, H, _ = q.shape
    G = k.shape[1]
    bucket = torch.tensor([distance_bucket(n, rel.shape[0], bias_max) for n in range(L)])
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for i in range(L):
        j0 = max(0, i - window + 1)
        bias = rel[bucket[i - torch.arange(j0, i + 1)]]
        for head in range(H):
            g = head // (H // G)
            s = (k[j0:i + 1, g] @ q[i, head]) * scale + bias[:, head]
            top = torch.maximum(s.max(), sink[head])
            e = torch.exp(s - top)
            out[i, head] = (e / (e.sum() + torch.exp(sink[head] - top))) @ v[j0:i + 1, g]
    return out


def left_mixer(h, w, p, m, eps):
    L, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w[p + "q"].T + w[p + "q.b"], w[p + "q.norm"], eps).reshape(L, H, d)
    k = rms_norm(h @ w[p + "k"].T + w[p + "k.b"], w[p + "k.norm"], eps).reshape(L, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(L, G, vd)
    o = windowed_attention(q, k, v, w[p + "rel"], w[p + "sink"], m["scale"], m["mask"]["size"], m["bias_max"])
    return o.reshape(L, H * vd) @ w[p + "o"].T


# ---------------------------------------------------------------------------------------------- gated delta rule
def causal_conv_silu(u, taps):
    """u (L, channels), taps (channels, n) the last column weighting the newest token; missing predecessors are zero."""
    L, n = u.shape[0], taps.shape[1]
    out = torch.zeros_like(u)
    for t in range(L):
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                out[t] += taps[:, j] * u[src]
    return silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def head_decay(a, A_log, dt_bias):
    return torch.exp(-torch.exp(A_log) * softplus(a + dt_bias))


def delta_scan(q, k, v, beta, g):
    """q, k (L, H, K), v (L, H, V), beta and g (L, H) -> read-outs (L, H, V) and the last state (H, K, V)."""
    L, H, K = q.shape
    S = torch.zeros(H, K, v.shape[2], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(L):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (k[t][:, :, None] * S).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (q[t][:, :, None] * S).sum(1)
    return out, S


def right_mixer(h, w, p, m, eps):
    L, H, G, K, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = lambda n: causal_conv_silu(h @ w[p + n].T, w[p + n + ".conv"])
    spread = lambda x: x.repeat_interleave(H // G, dim=1)
    q = spread(unit(conv("q").reshape(L, G, K)) * K ** -0.5)
    k = spread(unit(conv("k").reshape(L, G, K)))
    v = conv("v").reshape(L, H, V)
    beta = sigmoid(h @ w[p + "b"].T)
    g = head_decay(h @ w[p + "a"].T, w[p + "A_log"], w[p + "dt_bias"])
    o, _ = delta_scan(q, k, v, beta, g)
    o = rms_norm(o, w[p + "norm"], eps).reshape(L, H * V)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    left = left_mixer(h, w, p + "left.", m["left"], eps)
    right = right_mixer(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


# ---------------------------------------------------------------------------------------------- feed-forward
def dense(h, w, p, spec):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def clamped_glu(gate, up, limit):
    g = gate.clamp(max=limit)
    return g * sigmoid(1.702 * g) * (up.clamp(-limit, limit) + 1.0)


def expert(h, w, p, limit):
    return clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def route(z, top, groups=None):
    """Chosen experts (L, top), best first, and their weights, from router logits z (L, experts)."""
    s = torch.softmax(z, dim=-1)
    allowed = torch.ones_like(s, dtype=torch.bool)
    if groups:
        n, size = groups["count"], s.shape[1] // groups["count"]
        best = s.reshape(-1, n, size).amax(-1)
        kept = torch.zeros_like(best, dtype=torch.bool)
        kept.scatter_(1, best.argsort(dim=-1, descending=True)[:, :groups["keep"]], True)
        allowed = kept.repeat_interleave(size, dim=1)
    idx = torch.where(allowed, s, torch.full_like(s, -1.0)).argsort(dim=-1, descending=True, stable=True)[:, :top]
    weight = s.gather(1, idx)
    return idx, weight / (weight.sum(-1, keepdim=True) + 1e-20)


def moe(h, w, p, spec):
    idx, weight = route(h @ w[p + "router"].T, spec["router"]["top"], spec["router"].get("groups"))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(idx.shape[1]):
            out[t] += weight[t, k] * expert(h[t:t + 1], w, f"{p}e{int(idx[t, k])}.", spec["expert"]["limit"])[0]
    if spec.get("shared"):
        out = out + expert(h, w, p + "shared.", spec["shared"]["limit"])
    return out


# ---------------------------------------------------------------------------------------------- model
def forward(config, weights, token_ids, dtype=torch.float64, per_layer=None):
    """Logits (L, vocab).  `per_layer`, a list, receives the residual stream after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = rms_norm(w["embed"][torch.as_tensor(token_ids)], w["embed.norm"], eps)
    mixers = {"gla": gla, "parallel": parallel}
    feed_forwards = {"dense": dense, "moe": moe}
    for i, layer in enumerate(config["layers"]):
        l = f"l{i}."
        x = x + rms_norm(mixers[layer["type"]](x, w, l + "mix.", layer["mixer"], eps), w[l + "norm1"], eps)
        if layer.get("mlp"):
            x = x + rms_norm(feed_forwards[layer["mlp"]["kind"]](x, w, l + "mlp.", layer["mlp"]), w[l + "norm2"], eps)
        if per_layer is not None:
            per_layer.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def random_weights(config, seed=0, rank=5, buckets=10):
    """Checkpoint tensors of a configuration from a seed, bfloat16, with every mechanism visible in the output
    (projections of unit gain, norms around one, sinks around zero, biases of the size of the scores, decays between slow
    and fast, router logits far apart)."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (gain / math.sqrt(i))

    def around(n, mean, spread):
        return mean + spread * torch.randn(n, generator=g)

    W = config["width"]
    w = {"embed": torch.randn(config["vocab"], W, generator=g), "embed.norm": around(W, 1.0, 0.1),
         "head": mat(config["vocab"], W), "final.norm": around(W, 1.0, 0.1)}
    for i, layer in enumerate(config["layers"]):
        l, m = f"l{i}.", layer["mixer"]
        p = l + "mix."
        w[l + "norm1"] = around(W, 1.0, 0.1)
        if layer["type"] == "gla":
            H, K, V = m["heads"], m["dim"], m["vdim"]
            w.update({p + "q": mat(H * K, W), p + "k": mat(H * K, W), p + "v": mat(H * V, W), p + "g": mat(H * V, W),
                      p + "o": mat(W, H * V), p + "norm": around(V, 1.0, 0.1), p + "a1": mat(rank, W),
                      p + "a2": mat(H * K, rank), p + "a2.b": around(H * K, 2.0, 2.0)})
        else:
            a, b = m["left"], m["right"]
            H, G, d, vd = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "left."
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * vd)):
                w[q + n], w[q + n + ".b"] = mat(rows, W), around(rows, 0.0, 0.3)
            w.update({q + "q.norm": around(H * d, 1.5, 0.2), q + "k.norm": around(G * d, 1.5, 0.2),
                      q + "rel": torch.randn(buckets, H, generator=g), q + "sink": around(H, 1.0, 0.5),
                      q + "o": mat(W, H * vd), q + "out": around(W, 1.0, 0.1)})
            H, G, K, V = b["heads"], b["kv_heads"], b["dim"], b["vdim"]
            q = p + "right."
            for n, rows in (("q", G * K), ("k", G * K), ("v", H * V)):
                w[q + n], w[q + n + ".conv"] = mat(rows, W), mat(rows, b["conv"])
            w.update({q + "b": mat(H, W), q + "a": mat(H, W), q + "A_log": around(H, -1.0, 1.0),
                      q + "dt_bias": around(H, -2.0, 1.0), q + "norm": around(V, 1.0, 0.1), q + "g": mat(H * V, W),
                      q + "o": mat(W, H * V), q + "out": around(W, 1.0, 0.1)})
        e = layer.get("mlp")
        if not e:
            continue
        w[l + "norm2"] = around(W, 1.0, 0.1)
        p = l + "mlp."
        names = [("", e["ff"])] if e["kind"] == "dense" else \
            [(f"e{j}.", e["expert"]["ff"]) for j in range(e["router"]["experts"])]
        if e["kind"] == "moe":
            w[p + "router"] = mat(e["router"]["experts"], W, 3.0)
            if e.get("shared"):
                names.append(("shared.", e["shared"]["ff"]))
        for name, ff in names:
            w[p + name + "gate"], w[p + name + "up"], w[p + name + "down"] = mat(ff, W, 1.5), mat(ff, W, 1.5), mat(W, ff)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
