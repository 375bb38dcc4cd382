"""Small Surelorn configurations with random weights, and the comparison of an engine with the slow restatement in
plain_surelorn.py.  Used by the CPU and the B200 tests."""
import torch

import plain_surelorn as plain
from cogito_b200.models.surelorn import Surelorn, SurelornConfig, random_tensors
from cogito_b200.serve.stack import StackEngine


def mixer(heads, dim, vdim, q_rank, kv_rank, scale):
    return {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}


def layer(m, mlp, weights_of=None):
    e = {"type": "latent_attention", "mixer": m, "mlp": mlp}
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, identity=None, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if identity is not None:
        r["identity"] = identity
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    e = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        e["shared"] = {"ff": shared}
    return e


def config(width, vocab, layers, scale=3.0, eps=1e-5):
    return {"architecture": "Surelorn", "width": width, "vocab": vocab, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


def cases():
    a = mixer(3, 24, 40, 40, 72, 0.31)
    mixed = [layer(a, moe(24, 6, 3, 2, (4, 2), 40)), layer(mixer(2, 16, 8, 24, 48, 0.5), dense(56)), layer(a, moe(24, 6, 3, 2, (4, 2), 40), 0),
             layer(a, None), layer(a, None, 3), layer(a, moe(24, 6, 3, 2, (4, 2), 40), 2)]
    b = mixer(17, 20, 12, 33, 36, 0.2)
    odd = [layer(b, moe(30, 5, 2)), layer(b, dense(42)), layer(b, moe(30, 5, 2), 0)]
    c = mixer(40, 128, 64, 128, 512, 0.09)
    wide = [layer(c, moe(64, 70, 6, 2, (8, 3))), layer(c, dense(96))]
    d = mixer(20, 144, 96, 64, 256, 0.1)
    long_heads = [layer(d, dense(128)), layer(mixer(48, 32, 32, 64, 192, 0.2), moe(32, 8, 1, 0, (1, 1), 32))]
    return {"mixed": config(96, 101, mixed), "odd": config(130, 77, odd, 1.0, 1e-6), "wide": config(256, 120, wide, 0.5),
            "long_heads": config(136, 64, long_heads)}


def build(name, seed=0):
    d = cases()[name]
    cfg = SurelornConfig.from_dict(d)
    return d, cfg, random_tensors(cfg, seed)


def engine(cfg, tensors, device, dtype, slots=4, max_len=1024, pool=2048, **kw):
    return StackEngine(Surelorn(cfg, tensors, device, dtype), slots, max_len, pool_tokens=pool, **kw)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def portions(n, sizes):
    """Cuts n tokens into portions of the given sizes, repeated, the rest one by one at the end."""
    out, i, k = [], 0, 0
    while i < n:
        s = min(sizes[k % len(sizes)], n - i)
        out.append((i, s))
        i, k = i + s, k + 1
    return out


def feed(e, toks, cuts, slot=None):
    """All logits [T, V] of one sequence fed in the given portions."""
    own = slot is None
    if own:
        slot = e.open()
    out = [e.step([(slot, toks[i:i + n], list(range(n)))]) for i, n in cuts]
    if own:
        e.close(slot)
    return torch.cat(out).double().cpu()


def row_errors(got, want):
    """Root mean square over the vocabulary of the difference, over the logits' own scale."""
    return ((got - want) ** 2).mean(-1).sqrt() / want.std()


def expect(d, tensors, toks):
    return plain.forward(d, tensors, toks)


def assert_close(got, want, dtype, what=""):
    err = row_errors(got, want)
    if dtype == torch.float32:
        assert float(err.max()) < 1e-4, (what, float(err.max()))
    else:
        # bf16: a close call of a router may fall the other way at a few positions; those move a lot
        good = err < 0.06
        assert float(err.median()) < 0.03 and float(good.double().mean()) >= 0.9, (what, float(err.median()), float(err.max()))
