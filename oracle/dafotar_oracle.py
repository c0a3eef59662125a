"""Plain restatement of the Dafotar decoder on the CPU: one function per mechanism, written for reading, not for speed, and
sharing no code with the package.  A whole sequence goes in, position by position where the mechanism is recurrent; there is
no cache, no batching and no cutting into portions.

Notation: a sequence is an (L, width) matrix, weights are (out, in) and applied as `x @ W.T`.  `w` is a dict of tensors
under the checkpoint's names; everything is computed in the dtype of those tensors (float64 by default).
"""
import math

import torch


def sigmoid(z):
    return torch.exp(-torch.logaddexp(torch.zeros_like(z), -z))


def log_sigmoid(z):
    return -torch.logaddexp(torch.zeros_like(z), -z)


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def layer_norm(x, weight, bias, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


# ---------------------------------------------------------------------------------------------- streams and input convolution
def gather_streams(x, a):
    """x (streams, L, width), a (streams,) -> what a sublayer reads, before its norm."""
    u = torch.zeros_like(x[0])
    for s in range(x.shape[0]):
        u = u + a[s] * x[s]
    return u


def update_streams(x, y, mix, out):
    """Every new stream is a mixture of the old ones, mix[from, to], plus its share of the sublayer's result."""
    new = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for s in range(x.shape[0]):
            new[t] += mix[s, t] * x[s]
        new[t] += out[t] * y
    return new


def causal_conv(h, taps):
    """h (L, channels), taps (channels, n) the last column weighting the newest token; missing predecessors are zero."""
    L, n = h.shape[0], taps.shape[1]
    out = torch.zeros_like(h)
    for t in range(L):
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                out[t] += taps[:, j] * h[src]
    return out


# ---------------------------------------------------------------------------------------------- attention
def rotate(x, positions, base, dims):
    """x (L, heads, d): pairs (i, i + dims / 2) of the first `dims` entries turn by position * base^(-2 i / dims)."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = (positions * base ** (-2.0 * i / dims))[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + half] = v * torch.cos(a) + u * torch.sin(a)
    return out


def keys_values(h, w, p, m, eps):
    """Rotated keys (L, G, dim) and rotated values (L, G, vdim), as a later layer may use them too."""
    L, G, d, vd = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(L).to(h.dtype)
    k = rms_norm((h @ w[p + "k"].T).reshape(L, G, d), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T).reshape(L, G, vd)
    return rotate(k, pos, m["rot"]["base"], m["rot"]["dims"]), rotate(v, pos, m["rot"]["base"], vd)


def windowed_attention(q, k, v, factor, window):
    """q (L, H, d), k (L, G, d), v (L, G, vd), factor (H,) of the scores -> (L, H, vd)."""
    L, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for i in range(L):
        j0 = max(0, i - window + 1)
        for head in range(H):
            g = head // (H // G)
            s = (k[j0:i + 1, g] @ q[i, head]) * factor[head]
            e = torch.exp(s - s.max())
            out[i, head] = (e / e.sum()) @ v[j0:i + 1, g]
    return out


def attention(h, w, p, m, eps, kv=None):
    """Returns the result and the keys and values used (`kv`: those of an earlier layer)."""
    L, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = torch.arange(L).to(h.dtype)
    k, v = kv if kv is not None else keys_values(h, w, p, m, eps)
    q = rms_norm((h @ w[p + "q"].T).reshape(L, H, d), w[p + "q.norm"], eps)
    q = rotate(q, pos, m["rot"]["base"], m["rot"]["dims"])
    o = windowed_attention(q, k, v, m["scale"] * w[p + "temp"], m["mask"]["size"])
    o = rotate(o, -pos, m["rot"]["base"], vd)
    return o.reshape(L, H * vd) @ w[p + "o"].T, (k, v)


# ---------------------------------------------------------------------------------------------- matrix memory
def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def mlstm_scan(q, k, v, i, f):
    """q, k (L, H, K), v (L, H, V), i and f (L, H) logarithms of the gates.  Returns the read-outs (L, H, V) and the last
    state: S (H, K, V), n (H, K), m (H)."""
    L, H, K = q.shape
    S, n, m = torch.zeros(H, K, v.shape[2], dtype=q.dtype), torch.zeros(H, K, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(L):
        new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - new)[:, None], torch.exp(i[t] - new)[:, None]
        S = keep[:, :, None] * S + (write * k[t])[:, :, None] * v[t][:, None, :]
        n = keep * n + write * k[t]
        m = new
        weight = torch.maximum((n * q[t]).sum(1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (q[t][:, :, None] * S).sum(1) / weight[:, None]
    return out, (S, n, m)


def mlstm(h, w, p, m, eps):
    L, H, K, V, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).reshape(L, H, K) * K ** -0.5
    k = (h @ w[p + "k"].T).reshape(L, H, K)
    v = (h @ w[p + "v"].T).reshape(L, H, V)
    i = soft_cap(h @ w[p + "i"].T + w[p + "i.b"], cap)
    f = log_sigmoid(soft_cap(h @ w[p + "f"].T + w[p + "f.b"], cap))
    o, _ = mlstm_scan(q, k, v, i, f)
    o = rms_norm(o, 1.0, eps).reshape(L, H * V) * w[p + "norm"]
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---------------------------------------------------------------------------------------------- feed-forward
def dense(h, w, p):
    return ((h @ w[p + "gate"].T).clamp(min=0) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ---------------------------------------------------------------------------------------------- model
def forward(config, weights, token_ids, dtype=torch.float64, per_layer=None):
    """Logits (L, vocab).  `per_layer`, a list, receives the sum of the streams after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(token_ids)].expand(config["streams"], -1, -1)
    kept = {}
    for i, layer in enumerate(config["layers"]):
        l, m = f"l{i}.", layer["mixer"]
        h = layer_norm(gather_streams(x, w[l + "hc1.in"]), w[l + "norm1"], w[l + "norm1.b"], eps)
        h = h + causal_conv(h, w[l + "canon1"])
        if layer["type"] == "mlstm":
            y = mlstm(h, w, l + "mix.", m, eps)
        else:
            y, kept[i] = attention(h, w, l + "mix.", m, eps, kept[m["kv_from"]] if "kv_from" in m else None)
        x = update_streams(x, y, w[l + "hc1.mix"], w[l + "hc1.out"])
        if layer.get("mlp"):
            h = layer_norm(gather_streams(x, w[l + "hc2.in"]), w[l + "norm2"], w[l + "norm2.b"], eps)
            x = update_streams(x, dense(h, w, l + "mlp."), w[l + "hc2.mix"], w[l + "hc2.out"])
        if per_layer is not None:
            per_layer.append(x.sum(0))
    return layer_norm(x.sum(0), w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T


def random_weights(config, seed=0):
    """Checkpoint tensors of a configuration from a seed, bfloat16, with every mechanism visible in the output
    (projections of unit gain, norms around one, streams that differ, forget gates mostly open, input gates around
    minus one)."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (gain / math.sqrt(i))

    def around(n, mean, spread):
        return mean + spread * torch.randn(n, generator=g)

    W, S, taps = config["width"], config["streams"], config["canon"]["taps"]
    w = {"embed": torch.randn(config["vocab"], W, generator=g), "final.norm": around(W, 1.0, 0.1), "final.norm.b": around(W, 0.0, 0.1)}
    for i, layer in enumerate(config["layers"]):
        l, m = f"l{i}.", layer["mixer"]
        p = l + "mix."
        w[l + "canon1"] = torch.randn(W, taps, generator=g) * 0.5
        for q in (1, 2) if layer.get("mlp") else (1,):
            w[l + f"norm{q}"], w[l + f"norm{q}.b"] = around(W, 1.0, 0.1), around(W, 0.0, 0.1)
            w[l + f"hc{q}.in"], w[l + f"hc{q}.out"] = around(S, 1.0 / S, 0.3), around(S, 1.0, 0.3)
            w[l + f"hc{q}.mix"] = 0.9 * torch.eye(S) + 0.15 * torch.randn(S, S, generator=g)
        H, d, vd = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "mlstm":
            w.update({p + "q": mat(H * d, W), p + "k": mat(H * d, W), p + "v": mat(H * vd, W), p + "g": mat(H * vd, W),
                      p + "o": mat(W, H * vd), p + "norm": around(H * vd, 1.0, 0.1), p + "i": mat(H, W),
                      p + "i.b": around(H, -1.0, 1.0), p + "f": mat(H, W), p + "f.b": around(H, 3.0, 1.0)})
        else:
            w.update({p + "q": mat(H * d, W), p + "q.norm": around(d, 1.0, 0.2), p + "temp": around(H, 1.2, 0.3),
                      p + "o": mat(W, H * vd, 1.5)})
            if "kv_from" not in m:
                w.update({p + "k": mat(m["kv_heads"] * d, W), p + "v": mat(m["kv_heads"] * vd, W), p + "k.norm": around(d, 1.0, 0.2)})
        if layer.get("mlp"):
            p, ff = l + "mlp.", layer["mlp"]["ff"]
            w[p + "gate"], w[p + "up"], w[p + "down"] = mat(ff, W, 1.5), mat(ff, W, 1.5), mat(W, ff)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
