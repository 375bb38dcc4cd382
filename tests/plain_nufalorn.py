"""Slow restatement of the Nufalorn decoder, one function per mechanism, in the precision of its inputs (the tests pass
fp64).  It shares no code with the package: one sequence at a time, every head and every position by itself.

    x = E[tok];   x <- x + m (mixer(n1(x)) + ff(n2(x)));   out = cap tanh(head n_final(x) / cap)

n(.) scales by 1 + w.  Mixers: attention inside blocks of positions, with turned values and a sink; two linear
recurrences S <- diag(a) S + k v^T, o = S^T q that differ in where a, k and q come from.
"""
import math

import torch


def rms(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def turn(vec, position, base, dims, sign=1):
    """vec [.., D]: elements 2i and 2i + 1, 2i < dims, are a plane turned by sign * position * base^(-2i / dims)."""
    out = vec.clone()
    for i in range(dims // 2):
        a = sign * position * base ** (-2.0 * i / dims)
        c, s = math.cos(a), math.sin(a)
        u, v = vec[..., 2 * i], vec[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def keys_values(x, w, m, eps):
    """What the cache of an attention layer holds: keys and values [T, kv_heads, .] after all rotations."""
    T, G = x.shape[0], m["kv_heads"]
    k = (x @ w["k"].T).view(T, G, m["dim"])
    v = rms((x @ w["v"].T).view(T, G, m["vdim"]), eps)
    rot = m["rot"]
    k = torch.stack([turn(k[j], j, rot["base"], rot["dims"]) for j in range(T)])
    v = torch.stack([turn(v[j], j, rot["base"], m["vdim"]) for j in range(T)])
    return k, v


def visible(i, size):
    """Positions that position i sees: its own block's, up to itself."""
    return range(i // size * size, i + 1)


def sink_weights(scores):
    """exp(s_j) / (1 + sum exp(s)), written with the largest of all scores (the sink's is 0) taken out."""
    top = max(float(scores.max()), 0.0)
    e = torch.exp(scores - top)
    return e / (math.exp(-top) + e.sum())


def attention(x, w, m, k, v):
    """x [T, width]; keys and values may be another layer's."""
    T, H, G, rot = x.shape[0], m["heads"], m["kv_heads"], m["rot"]
    q = (x @ w["q"].T).view(T, H, m["dim"])
    out = torch.zeros(T, H, m["vdim"], dtype=x.dtype)
    for i in range(T):
        qi = turn(q[i], i, rot["base"], rot["dims"])
        see = visible(i, m["mask"]["size"])
        lo, hi = see.start, see.stop
        for h in range(H):
            g = h // (H // G)
            p = sink_weights(k[lo:hi, g] @ qi[h] * m["scale"])
            out[i, h] = p @ v[lo:hi, g]
        out[i] = turn(out[i], i, rot["base"], m["vdim"], -1)
    return out.reshape(T, -1) @ w["o"].T


def recurrence(q, k, v, a):
    """q, k, a [T, H, D], v [T, H, V] -> o [T, H, V]; state rows belong to the elements of q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def hgrn2(x, w, m, eps):
    T, shape = x.shape[0], (x.shape[0], m["heads"], m["dim"])
    low = w["lower"]
    f = low + (1 - low) * sigmoid(x @ w["f"].T + w["f.b"])
    q, f = silu(x @ w["q"].T).view(shape), f.view(shape)
    o = recurrence(q, 1 - f, (x @ w["v"].T).view(T, m["heads"], m["vdim"]), f)
    return (rms(o, eps) * w["norm"]).reshape(T, -1) @ w["o"].T


def gla(x, w, m, eps):
    T, shape = x.shape[0], (x.shape[0], m["heads"], m["dim"])
    z = (x @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    a = sigmoid(z) ** (1.0 / m["tau"])
    q, k = (x @ w["q"].T).view(shape) * m["dim"] ** -0.5, (x @ w["k"].T).view(shape)
    o = recurrence(q, k, (x @ w["v"].T).view(T, m["heads"], m["vdim"]), a.view(shape))
    return ((rms(o, eps) * w["norm"]).reshape(T, -1) * silu(x @ w["g"].T)) @ w["o"].T


def feed_forward(x, w):
    return (torch.clamp(x @ w["gate"].T, min=0) * (x @ w["up"].T)) @ w["down"].T


def forward(cfg, weights, tokens, dtype=torch.float64, keep=None):
    """Logits [T, vocab] of one sequence; keep: a list that receives the residual after every layer."""
    eps, mult, cap = cfg["norm"]["eps"], cfg["residual_mult"], cfg["logit_softcap"]
    w = {k: v.to(dtype) for k, v in weights.items()}
    x = w["embed"][torch.tensor(tokens)]
    kv = {}
    for i, layer in enumerate(cfg["layers"]):
        m = layer["mixer"]

        def sub(part):
            return {k[len(f"l{i}.{part}."):]: v for k, v in w.items() if k.startswith(f"l{i}.{part}.")}
        h, t = rms(x, eps) * (1 + w[f"l{i}.norm1"]), sub("mix")
        if layer["type"] == "attention":
            home = m.get("kv_from", i) if m.get("kv_from") is not None else i
            if home == i:
                kv[i] = keys_values(h, t, m, eps)
            y = attention(h, t, m, *kv[home])
        else:
            y = {"hgrn2": hgrn2, "gla": gla}[layer["type"]](h, t, m, eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(rms(x, eps) * (1 + w[f"l{i}.norm2"]), sub("mlp"))
        x = x + mult * y
        if keep is not None:
            keep.append(x.clone())
    logits = (rms(x, eps) * (1 + w["final.norm"])) @ w["head"].T
    return cap * torch.tanh(logits / cap)
