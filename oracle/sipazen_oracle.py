"""Plain restatement of the Sipazen decoder on the CPU: one function per mechanism, written for reading, not for
speed, and sharing no code with the package.  A whole sequence goes in, position by position where the mechanism
is recurrent; there is no cache, no batching and no cutting into portions.

Notation: a sequence is an (L, width) matrix, weights are (out, in) and applied as `x @ W.T`.  `w` is a dict of
tensors under the checkpoint's names; everything is computed in the dtype of those tensors (float64 by default).
"""
import math

import torch


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.where(z > 0, z + torch.log1p(torch.exp(-z.abs())), torch.log1p(torch.exp(-z.abs())))


def grouped_rms_norm(x, weight, groups, eps):
    """x of every token cut into `groups` runs of equal length, each normalised by itself, then scaled by `weight`."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    parts = parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)
    return parts.reshape(x.shape) * weight


def rotate(x, position, base, dims):
    """Rotate-half rotary embedding of the first `dims` entries of the last dimension of x at one position."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = torch.tensor(position * base ** (-2.0 * i / dims), dtype=x.dtype)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + half] = v * torch.cos(a) + u * torch.sin(a)
    return out


def latent_attention(h, w, p, m, eps):
    """h (L, width), tensors w[p + name], m = the layer's mixer sizes.  Returns (L, width)."""
    L = h.shape[0]
    H, d, r, vd, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = (h @ w[p + "q"].T).reshape(L, H, d + r)
    down = h @ w[p + "dkv"].T
    c = grouped_rms_norm(down[:, :rank], w[p + "dkv.norm"], 1, eps)
    kr = torch.stack([rotate(down[t, rank:], t, base, dims) for t in range(L)])
    qr = torch.stack([rotate(q[t, :, d:], t, base, dims) for t in range(L)])
    k = (c @ w[p + "uk"].T).reshape(L, H, d)
    v = (c @ w[p + "uv"].T).reshape(L, H, vd)
    out = torch.zeros(L, H, vd, dtype=h.dtype)
    for t in range(L):
        for head in range(H):
            s = (k[:t + 1, head] @ q[t, head, :d] + kr[:t + 1] @ qr[t, head]) * m["scale"]
            sink = w[p + "sink"][head]
            top = torch.maximum(s.max(), sink)
            e = torch.exp(s - top)
            out[t, head] = (e / (e.sum() + torch.exp(sink - top))) @ v[:t + 1, head]
    gated = out.reshape(L, H * vd) * sigmoid(h @ w[p + "g"].T)
    return gated @ w[p + "o"].T


def causal_conv_silu(u, taps, bias):
    """u (L, channels), taps (channels, n) the last column weighting the newest token; missing predecessors count as zero."""
    L, n = u.shape[0], taps.shape[1]
    out = torch.zeros_like(u)
    for t in range(L):
        acc = bias.clone()
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                acc = acc + taps[:, j] * u[src]
        out[t] = silu(acc)
    return out


def ssm_scan(x, B, C, dt, A_log, D):
    """x (L, heads, P), B and C (L, groups, N), dt (L, heads) already positive.  Returns y (L, heads, P) and the
    final state (heads, N, P)."""
    L, H, P = x.shape
    per = H // B.shape[1]
    S = torch.zeros(H, B.shape[2], P, dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(L):
        for head in range(H):
            g = head // per
            S[head] = torch.exp(-torch.exp(A_log[head]) * dt[t, head]) * S[head] + \
                dt[t, head] * torch.outer(B[t, g], x[t, head])
            y[t, head] = S[head].T @ C[t, g] + D[head] * x[t, head]
    return y, S


def mamba2(h, w, p, m, eps):
    L = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    u = h @ w[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = causal_conv_silu(xbc, w[p + "conv"], w[p + "conv.b"])
    x = xbc[:, :inner].reshape(L, H, P)
    B = xbc[:, inner:inner + G * N].reshape(L, G, N)
    C = xbc[:, inner + G * N:].reshape(L, G, N)
    y, _ = ssm_scan(x, B, C, softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    y = grouped_rms_norm(y.reshape(L, inner) * silu(z), w[p + "norm"], m["norm_groups"], eps)
    return y @ w[p + "o"].T


def swiglu(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, W, b, top):
    """Chosen experts (L, top), best first, and mixing weights that sum to one over the chosen set."""
    z = h @ W.T + b
    best, idx = torch.sort(z, dim=-1, descending=True)
    best, idx = best[:, :top], idx[:, :top]
    e = torch.exp(best - best[:, :1])
    return idx, e / e.sum(-1, keepdim=True)


def moe(h, w, p, spec):
    idx, weight = route(h, w[p + "router"], w[p + "router.b"], spec["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(idx.shape[1]):
            out[t] += weight[t, k] * swiglu(h[t:t + 1], w, f"{p}e{int(idx[t, k])}.")[0]
    if spec.get("shared"):
        out = out + sigmoid(h @ w[p + "shared.sg"].T) * swiglu(h, w, p + "shared.")
    return out


def forward(config, weights, token_ids, dtype=torch.float64, per_layer=None):
    """Logits (L, vocab).  `per_layer`, a list, receives the residual stream after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    groups, eps, mult = config["norm"]["groups"], config["norm"]["eps"], config["residual_mult"]
    x = w["embed"][torch.as_tensor(token_ids)]
    mixers = {"mamba2": mamba2, "latent_attention": latent_attention}
    for i, layer in enumerate(config["layers"]):
        l = f"l{i}."
        h = grouped_rms_norm(x, w[l + "norm1"], groups, eps)
        y = mixers[layer["type"]](h, w, l + "mix.", layer["mixer"], eps)
        y = y * sigmoid(h @ w[l + "rg1"].T + w[l + "rg1.b"])
        x = x + mult * grouped_rms_norm(y, w[l + "norm1b"], groups, eps)
        if layer.get("mlp"):
            h = grouped_rms_norm(x, w[l + "norm2"], groups, eps)
            y = moe(h, w, l + "mlp.", layer["mlp"]) * sigmoid(h @ w[l + "rg2"].T + w[l + "rg2.b"])
            x = x + mult * grouped_rms_norm(y, w[l + "norm2b"], groups, eps)
        if per_layer is not None:
            per_layer.append(x)
    return grouped_rms_norm(x, w["final.norm"], groups, eps) @ w["head"].T


def random_weights(config, seed=0, scale=1.0):
    """Checkpoint tensors of a configuration from a seed, bfloat16, with every mechanism visible in the output
    (projections of unit gain, norms around one, sinks around zero, decays between slow and fast)."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (gain / math.sqrt(i))

    def around(n, mean, spread):
        return mean + spread * torch.randn(n, generator=g)

    W = config["width"]
    w = {"embed": torch.randn(config["vocab"], W, generator=g), "head": mat(config["vocab"], W),
         "final.norm": around(W, 1.0, 0.1)}
    for i, layer in enumerate(config["layers"]):
        l, m = f"l{i}.", layer["mixer"]
        p = l + "mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer.get("mlp") else ()):
            w[l + n] = around(W, 1.0, 0.1)
        for n in ("rg1",) + (("rg2",) if layer.get("mlp") else ()):
            w[l + n], w[l + n + ".b"] = mat(W, W), around(W, 0.5, 0.3)
        if layer["type"] == "latent_attention":
            H, d, r, vd, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w.update({p + "q": mat(H * (d + r), W, 1.5 * scale), p + "dkv": mat(rank + r, W), p + "dkv.norm": around(rank, 1.0, 0.1),
                      p + "uk": mat(H * d, rank, 1.5), p + "uv": mat(H * vd, rank), p + "sink": around(H, 1.0, 0.5),
                      p + "g": mat(H * vd, W), p + "o": mat(W, H * vd)})
        else:
            H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            ch = H * P + 2 * G * N
            w.update({p + "in": mat(H * P + ch + H, W), p + "conv": mat(ch, m["conv"]), p + "conv.b": around(ch, 0.0, 0.2),
                      p + "dt_bias": around(H, -1.0, 1.0), p + "A_log": around(H, -1.0, 1.0), p + "D": around(H, 1.0, 0.3),
                      p + "norm": around(H * P, 1.0, 0.1), p + "o": mat(W, H * P)})
        if layer.get("mlp"):
            p, e = l + "mlp.", layer["mlp"]
            n = e["router"]["experts"]
            w[p + "router"], w[p + "router.b"] = mat(n, W), around(n, 0.0, 1.5)
            names = [(f"e{j}.", e["expert"]["ff"]) for j in range(n)]
            if e.get("shared"):
                names.append(("shared.", e["shared"]["ff"]))
                w[p + "shared.sg"] = mat(1, W)
            for name, ff in names:
                w[p + name + "gate"], w[p + name + "up"] = mat(ff, W, 1.5), mat(ff, W, 1.5)
                w[p + name + "down"] = mat(W, ff)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
