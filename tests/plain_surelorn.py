"""Slow restatement of the Surelorn decoder, one function per mechanism, in the precision of its inputs
(the tests pass fp64).  It shares no code with the package: plain tensors in, plain tensors out, one
sequence at a time, every key of every head expanded, experts visited one token at a time.

    x_0   = s * E[tok] + pos(p)                      pos: sin / cos pairs, frequency 10000^(-2i / width)
    x    <- x + n1(attention(x));  x <- x + n2(feed_forward(x))        n(.): RMS norm with a weight
    out   = head @ n_final(x)
"""
import math

import torch


def rms(v, w, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * w


def sinusoid(positions, width, dtype=torch.float64):
    out = torch.zeros(len(positions), width, dtype=torch.float64)
    for row, p in enumerate(positions):
        for j in range(width):
            angle = float(p) * 10000.0 ** (-2.0 * (j // 2) / width)
            out[row, j] = math.sin(angle) if j % 2 == 0 else math.cos(angle)
    return out.to(dtype)


def silu(z):
    return z / (1 + torch.exp(-z))


def gated(x, gate, up, down):
    return (silu(x @ gate.T) * (x @ up.T)) @ down.T


def latent_attention(x, w, m, eps):
    """x [T, width]; w: the mixer's tensors by short name; m: its sizes.  All T tokens of one sequence."""
    T, H, d, v = x.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (rms(x @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).view(T, H, d)
    c = rms(x @ w["dkv"].T, w["dkv.norm"], eps)
    k = (c @ w["uk"].T).view(T, H, d)
    val = (c @ w["uv"].T).view(T, H, v)
    out = torch.zeros(T, H, v, dtype=x.dtype)
    for h in range(H):
        score = (q[:, h] @ k[:, h].T) * m["scale"]
        for i in range(T):
            row = score[i, :i + 1]
            e = torch.exp(row - row.max())
            out[i, h] = (e / e.sum()) @ val[:i + 1, h]
    return out.reshape(T, H * v) @ w["o"].T


def choose(logits, correction, router):
    """logits [outputs] of one token -> [(output index, weight)], best choice score first."""
    e = torch.exp(logits - logits.max())
    s = e / e.sum()
    choice = s + correction
    n = len(s)
    allowed = set(range(n))
    g = router.get("groups")
    if g:
        per = n // g["count"]
        best = [(max(float(choice[i * per + j]) for j in range(per)), -i) for i in range(g["count"])]
        kept = [-neg for _, neg in sorted(best, reverse=True)[:g["keep"]]]
        allowed = {i * per + j for i in kept for j in range(per)}
    picked = sorted(allowed, key=lambda i: (-float(choice[i]), i))[:router["top"]]
    total = sum(s[i] for i in picked) + 1e-20
    return [(i, s[i] / total) for i in picked]


def mixture(x, w, mlp):
    router = mlp["router"]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for i, weight in choose(w["router"] @ x[t], w["correction"], router):
            if i < router["experts"]:
                y = gated(x[t:t + 1], w[f"e{i}.gate"], w[f"e{i}.up"], w[f"e{i}.down"])[0]
            else:
                y = x[t]
            out[t] += weight * y
        if mlp.get("shared"):
            out[t] += gated(x[t:t + 1], w["shared.gate"], w["shared.up"], w["shared.down"])[0]
    return out


def home_layer(layers, i):
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg, weights, tokens, dtype=torch.float64, keep=None):
    """Logits [T, vocab] of one sequence; keep: a list that receives the residual after every layer."""
    eps = cfg["norm"]["eps"]
    w = {k: v.to(dtype) for k, v in weights.items()}
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"] + sinusoid(range(len(tokens)), cfg["width"], dtype)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{home_layer(cfg['layers'], i)}."

        def sub(part):
            return {k[len(p + part):]: v for k, v in w.items() if k.startswith(p + part)}
        x = x + rms(latent_attention(x, sub("mix."), layer["mixer"], eps), w[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            s = sub("mlp.")
            y = gated(x, s["gate"], s["up"], s["down"]) if mlp["kind"] == "dense" else mixture(x, s, mlp)
            x = x + rms(y, w[p + "norm2"], eps)
        if keep is not None:
            keep.append(x.clone())
    return rms(x, w["final.norm"], eps) @ w["head"].T
