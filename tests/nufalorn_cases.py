"""Small Nufalorn configurations with random weights, and the comparison of an engine with the slow restatement in
plain_nufalorn.py.  Used by the CPU and the B200 tests."""
import torch

import plain_nufalorn as plain
from cogito_b200.models.nufalorn import Nufalorn, NufalornConfig, random_tensors
from cogito_b200.serve.stack import StackEngine


def attention(heads, kv_heads, dim, vdim, scale, block, base=5000.0, rot=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": block},
         "rot": {"base": base, "dims": dim if rot is None else rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def hgrn2(heads, dim, vdim):
    return "hgrn2", {"heads": heads, "dim": dim, "vdim": vdim}


def gla(heads, dim, vdim, tau, a_rank):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "a_rank": a_rank}


def config(width, vocab, layers, mult=0.7, cap=12.0, eps=1e-5):
    """layers: ((kind, mixer), ff or None)."""
    out = [{"type": k, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (k, m), ff in layers]
    return {"architecture": "Nufalorn", "width": width, "vocab": vocab, "residual_mult": mult, "logit_softcap": cap, "norm": {"eps": eps}, "layers": out}


def cases():
    mixed = [(attention(6, 2, 24, 40, 0.3, 37, rot=16), 56), (hgrn2(3, 16, 24), 40), (gla(2, 40, 16, 4.0, 8), None),
             (attention(4, 2, 24, 40, 0.5, 50, base=300.0, rot=8, kv_from=0), 56), (gla(1, 24, 32, 1.0, 24), 24)]
    # the second attention layer reads the first one's cache: its rotation is the same
    mixed[3][0][1]["rot"] = dict(mixed[0][0][1]["rot"])
    odd = [(hgrn2(3, 10, 6), 35), (attention(5, 5, 18, 10, 0.25, 7, rot=6), 35), (gla(1, 13, 7, 2.5, 5), 30), (attention(10, 5, 18, 10, 0.4, 1, rot=6, kv_from=1), None)]
    wide = [(attention(16, 2, 128, 128, 0.09, 64), 96), (hgrn2(2, 128, 128), 128), (gla(2, 64, 128, 12.0, 24), 64), (attention(3, 1, 64, 32, 0.2, 129, 2e5, 32), 64)]
    long_heads = [(attention(2, 1, 144, 160, 0.1, 90), 128), (hgrn2(1, 136, 200), 64), (gla(2, 8, 264, 16.0, 12), 64), (attention(2, 1, 32, 96, 0.2, 1000), 64)]
    return {"mixed": config(96, 101, mixed), "odd": config(90, 77, odd, 1.0, 25.0, 1e-6), "wide": config(256, 120, wide, 0.5, 20.0),
            "long_heads": config(136, 64, long_heads)}


def build(name, seed=0):
    d = cases()[name]
    cfg = NufalornConfig.from_dict(d)
    return d, cfg, random_tensors(cfg, seed)


def engine(cfg, tensors, device, dtype, slots=4, max_len=1024, pool=2048, **kw):
    return StackEngine(Nufalorn(cfg, tensors, device, dtype), slots, max_len, pool_tokens=pool, **kw)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def portions(n, sizes):
    """Cuts n tokens into portions of the given sizes, repeated."""
    out, i, k = [], 0, 0
    while i < n:
        s = min(sizes[k % len(sizes)], n - i)
        out.append((i, s))
        i, k = i + s, k + 1
    return out


def singles(lo, hi):
    return [(i, 1) for i in range(lo, hi)]


def feed(e, toks, cuts, slot=None):
    """All logits [T, V] of one sequence fed in the given portions."""
    own = slot is None
    if own:
        slot = e.open()
    out = [e.step([(slot, toks[i:i + n], list(range(n)))]) for i, n in cuts]
    if own:
        e.close(slot)
    return torch.cat(out).double().cpu()


def expect(d, tensors, toks):
    return plain.forward(d, tensors, toks)


def greedy(d, tensors, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(expect(d, tensors, seq)[-1].argmax()))
    return seq[len(prompt):]


def assert_close(got, want, dtype, what=""):
    """Root mean square over the vocabulary of the difference, over the logits' own scale."""
    err = ((got - want) ** 2).mean(-1).sqrt() / want.std()
    worst = int(err.argmax())
    assert float(err.max()) < (1e-4 if dtype == torch.float32 else 0.06), (what, worst, float(err.max()), float(err.median()))


def standing_out(n, dim, at, seed=0):
    """Keys [n, dim] of small random numbers with one, at position ``at``, that a query along it finds, and that query."""
    g = torch.Generator().manual_seed(seed + n + at)
    k = torch.randn(n, dim, generator=g, dtype=torch.float64) * 0.1
    d = torch.randn(dim, generator=g, dtype=torch.float64)
    k[at] = d / d.norm() * 3
    return k, d / d.norm() * 3
