"""Nufalorn beside Surelorn and Llama at equal size (random weights): prompt and decode throughput, and a table of kernels.

    python benchmarks/nufalorn.py [--size 2048|4096|all] [--part model|kernels|all] [--iters 20] [--alone]

``model``: tokens/s of a prompt batch (hidden states and the logits of the last position) and of decoding one token per
sequence at a context of 2048, beside the framework's Surelorn (dense, bf16, same engine) and Llama (bf16 prompts, INT4
decoding) of the same width, feed-forward size and depth.  Decode steps are CUDA-graph replays.
``kernels``: each kernel of a Nufalorn step on the shapes of that size and the like kernel of a Surelorn or Llama step
(``like`` names it): device time (median, L2 flushed by a 256 MiB write between calls, graph replay), the time its bytes or
FLOPs need at the measured peaks, and the ratio of the two.  --alone leaves the other models out.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "benchmarks"))

import surelorn as other                                       # noqa: E402

SIZES = {2048: dict(heads=16, kv_heads=4, dim=128, ff=5632, layers=8), 4096: dict(heads=32, kv_heads=8, dim=128, ff=11008, layers=8)}
VOCAB, CONTEXT, BLOCK, RANK = other.VOCAB, other.CONTEXT, 4096, 32
BF, F32 = torch.bfloat16, torch.float32
ORDER = ("gla", "attention", "hgrn2", "gla", "hgrn2", "attention", "gla", "hgrn2")


def nufalorn_config(width, s):
    from cogito_b200.models.nufalorn import NufalornConfig
    H, d = s["heads"], s["dim"]
    kinds = {"attention": {"heads": H, "kv_heads": s["kv_heads"], "dim": d, "vdim": d, "scale": d ** -0.5, "mask": {"size": BLOCK}, "rot": {"base": 5e5, "dims": d}},
             "hgrn2": {"heads": H, "dim": d, "vdim": d}, "gla": {"heads": H, "dim": d, "vdim": d, "tau": 8.0, "a_rank": RANK}}
    layers = []
    for i, k in enumerate(ORDER):
        m = dict(kinds[k])
        if k == "attention" and i > ORDER.index(k):
            m["kv_from"] = ORDER.index(k)
        layers.append({"type": k, "mixer": m, "mlp": {"kind": "dense", "ff": s["ff"]}})
    return NufalornConfig.from_dict({"vocab": VOCAB, "width": width, "residual_mult": 0.8, "logit_softcap": 40.0, "norm": {"eps": 1e-5}, "layers": layers})


def model_part(width, iters=10, prompts=((1, 2048), (4, 2048), (1, 8192)), batches=(1, 16, 64), alone=False):
    """Every timed region streams more weights than L2 holds."""
    from cogito_b200.models.nufalorn import Nufalorn, random_tensors
    from cogito_b200.serve.stack import Segment, StackEngine, TokenBatch
    s, dev = SIZES[width], torch.device("cuda")
    out = {"width": width, **{k: s[k] for k in ("heads", "kv_heads", "layers", "ff")}, "context": CONTEXT}
    cfg = nufalorn_config(width, s)
    model = Nufalorn(cfg, random_tensors(cfg, 0, dev), dev, BF)
    rec = {"params": model.num_params()}
    for B, T in prompts:
        e = StackEngine(model, B, T)
        ids = torch.randint(0, VOCAB, (B, T), device=dev)

        def prompt():
            pos = torch.arange(T, device=dev, dtype=torch.int32).repeat(B)
            slot = torch.arange(B, device=dev, dtype=torch.int32).repeat_interleave(T)
            first = torch.arange(0, B * T, T, device=dev, dtype=torch.int32)
            b = TokenBatch(ids.view(-1), pos, slot, [Segment(0, B, T, 0, 0)], B * T, T, torch.stack([first, torch.full_like(first, T)], 1))
            return model.logits(model.stream(b, e.cache), torch.arange(T - 1, B * T, T, device=dev))
        with torch.no_grad():
            ms = other._timed(prompt, iters)
        rec[f"prompt_{B}x{T}"] = {"ms": round(ms, 3), "tok_per_s": round(B * T / ms * 1e3)}
        del e
    for B in batches:
        e = StackEngine(model, B, CONTEXT + 64)
        e.cache.lengths.fill_(CONTEXT)
        e._fresh = False
        tok = torch.randint(0, VOCAB, (B, 1), device=dev)
        ms = other._timed(other._graph(lambda: e.forward(tok)), iters)
        rec[f"decode_{B}"] = {"ms": round(ms, 3), "tok_per_s": round(B / ms * 1e3)}
        del e
        torch.cuda.empty_cache()
    out["nufalorn"] = rec
    del model
    torch.cuda.empty_cache()
    if not alone:
        rest = other.model_part(width, iters, batches=batches, kinds=("dense",))
        out.update({k: rest[k] for k in ("surelorn_dense", "llama")})
    return out


def kernel_part(width, iters=20, alone=False):
    from types import SimpleNamespace

    from kernels import Timer, peaks
    from cogito_b200.ops import misc as M
    from cogito_b200.ops import recurrence as R
    from cogito_b200.ops import rotary
    from cogito_b200.ops import stream as X
    from cogito_b200.ops.attention import flash_forward
    from cogito_b200.ops.linear import gated_linear, linear
    from cogito_b200.serve.hybrid_cache import HybridCache, KvShape
    hbm, tf, src = peaks()
    s, t, rows = SIZES[width], Timer(iters, 3), []
    H, G, D, ff = s["heads"], s["kv_heads"], s["dim"], s["ff"]
    mk = lambda *shape, dt=BF: torch.randn(*shape, device="cuda").to(dt)

    def put(name, like, fn, bytes_=0, flops=0, **extra):
        ms = t(fn, graph=True)
        floor = max(bytes_ / hbm / 1e6, flops / tf / 1e9)
        rows.append({"kernel": name, "like": like, "us": round(ms * 1e3, 2), "roofline_us": round(floor * 1e3, 2),
                     "fraction": round(floor / ms, 3), "bound": "hbm" if bytes_ / hbm / 1e6 >= flops / tf / 1e9 else "tensor", **extra})

    def product(name, like, M_, N_, K_, out=BF):
        a, b = mk(M_, K_), mk(N_, K_)
        put(name, like, lambda: linear(a, b, out_dtype=out), 2 * (M_ * K_ + N_ * K_) + (4 if out == F32 else 2) * M_ * N_, 2.0 * M_ * N_ * K_, shape=[M_, N_, K_])

    def recurrence(B, T, mode):
        """(rule, operands, states, batch, out) of B sequences of T tokens."""
        N = B * T
        rule = R.StateRule(H, D, D, mode, 1e-5, q_silu=mode == R.BOUNDED, q_scale=1.0 if mode == R.BOUNDED else D ** -0.5, tau=8.0)
        wide = mk(N, (2 if mode == R.BOUNDED else 4) * H * D)
        c = [wide[:, i * H * D:(i + 1) * H * D] for i in range(wide.shape[1] // (H * D))]
        z, bias = mk(N, H * D, dt=F32), 2 + mk(H * D, dt=F32)
        low = 0.9 * torch.rand(H * D, device="cuda") if mode == R.BOUNDED else None
        x = R.Operands(c[0], None, c[1], None, z, bias, low, 1 + mk(D, dt=F32)) if mode == R.BOUNDED else R.Operands(c[0], c[1], c[2], c[3], z, bias, None, 1 + mk(D, dt=F32))
        pos = torch.arange(T, device="cuda", dtype=torch.int32).repeat(B) if T > 1 else torch.full((B,), CONTEXT, device="cuda", dtype=torch.int32)
        slot = torch.arange(B, device="cuda", dtype=torch.int32).repeat_interleave(T)
        first = torch.arange(0, N, T, device="cuda", dtype=torch.int32)
        prompts = [SimpleNamespace(start=0, sequences=B, count=T, slot=0, begin=0)] if T > 1 else []
        batch = SimpleNamespace(slot=slot, pos=pos, runs=torch.stack([first, torch.full_like(first, T)], 1) if T > 1 else None, prompts=prompts, memo={})
        state = mk(B, 1, H, D, D, dt=F32)
        out = torch.empty(N, H * D + ff, dtype=BF, device="cuda")[:, :H * D]
        per_token = H * D * (2 + 2 + 4 + 2) if mode == R.BOUNDED else H * D * (2 * 4 + 4 + 2)
        flops = N * H * 2.0 * (2 * D * D + 32 * 2 * D) if T > 1 else 0        # state update, state read, 64-token triangle
        return (rule, x, state, batch, out), N * per_token + B * H * D * D * 4 * (1 if T > 1 else 2), flops

    with torch.no_grad():
        one = torch.zeros(1, device="cuda")
        put("smallest launch (what the method itself costs)", "-", lambda: one.add_(1))
        T = 4096
        # ---- prompt
        x, y, w = mk(T, width, dt=F32), mk(T, width), torch.ones(width, device="cuda")
        put("stream_norms (add, two norms)", "stream_update", lambda: X.stream_norms(x, 1e-5, BF, w, w, y=y, mult=0.5), T * width * (2 + 4 + 4 + 2 + 2))
        ids, table = torch.randint(0, VOCAB, (T,), device="cuda"), mk(VOCAB, width)
        put("stream_norms (embedding, two norms)", "embed_sinusoid", lambda: X.stream_norms(x, 1e-5, BF, w, w, ids=ids, table=table), T * width * (2 + 4 + 2 + 2))
        pos, slot = torch.arange(T, device="cuda", dtype=torch.int32), torch.zeros(T, device="cuda", dtype=torch.int32)
        freq = rotary.frequencies(5e5, D, "cuda")
        put("rotary_angles", "embed_sinusoid", lambda: rotary.angles(pos, freq), T * D * 4)
        cs = rotary.angles(pos, freq)
        cache = HybridCache([KvShape(G, D, D)], 1, T, 64, "cuda", BF)
        qkv = mk(T, (H + 2 * G) * D)
        q, k, v = qkv[:, :H * D], qkv[:, H * D:(H + G) * D], qkv[:, (H + G) * D:]
        put("kv_rotate_append", "latent_norm_append", lambda: cache.rotate_append(0, q, k, v, cs, cs, H, D, slot, pos, 1e-5, True), T * D * (4 * H + 12 * G + 8))
        put("kv_gather", "latent_gather", lambda: cache.gather(0, 0, 0, T, D), T * G * D * 8)
        qr, kr, vr = cache.rotate_append(0, q, k, v, cs, cs, H, D, slot, pos, 1e-5, True)
        heads = torch.empty(T, H * D + ff, dtype=BF, device="cuda")
        half = T // 2
        for name, blk in (("whole context", 0), ("blocks of 512", 512)):
            keys = half * half / 2 if not blk else half * blk / 2
            put(f"flash attention, {name}, sink, turned (2 x {half})", "flash attention",
                lambda: flash_forward(qr.view(2, half, H, D), kr.view(2, half, G, D), vr.view(2, half, G, D), causal=True, block=blk, sink=True, turn=cs.view(2, half, D // 2, 2),
                                      out=heads[:, :H * D].view(2, half, H, D)), T * D * (4 * H + 4 * G + 4), 2 * 4.0 * H * D * keys)
        for mode, name in ((R.BOUNDED, "hgrn2"), (R.ROOT, "gla")):
            for B, n in ((2, 2048), (1, 8192), (16, 1024)):
                args, by, fl = recurrence(B, n, mode)
                put(f"recurrence in chunks, {name} ({B} x {n})", "flash attention", lambda: R.advance(*args), by, fl)
                del args
        gu = mk(T, 2 * ff)
        put("gated rows (relu)", "swiglu", lambda: M.gated(gu, "relu", heads[:, H * D:]), T * ff * 6)
        product("gemm q|k|v", "gemm", T, (H + 2 * G) * D, width)
        product("gemm q|k|v|gate|decay", "gemm", T, 4 * H * D + RANK, width)
        product("gemm forget gate (fp32 out)", "gemm", T, H * D, width, F32)
        product("gemm decay (fp32 out)", "gemm", T, H * D, RANK, F32)
        product("gemm gate|up", "gemm", T, 2 * ff, width)
        product("gemm o|down", "gemm", T, width, H * D + ff)
        # ---- decode
        for B in (1, 16, 64):
            product(f"decode gemm q|k|v|gate|decay ({B})", "decode gemm", B, 4 * H * D + RANK, width)
            product(f"decode gemm decay ({B})", "decode gemm", B, H * D, RANK, F32)
            product(f"decode gemm o|down ({B})", "decode gemm", B, width, H * D + ff)
            product(f"decode gemm head ({B})", "decode gemm", B, VOCAB, width, F32)
            logits = mk(B, VOCAB, dt=F32)
            put(f"softcap ({B})", "decode norm", lambda: X.softcap(logits, 30.0), B * VOCAB * 8)
            ag, wg, act = mk(B, width), mk(2 * ff, width), torch.empty(B, H * D + ff, dtype=BF, device="cuda")
            put(f"decode gate|up with relu ({B})", "decode gate|up", lambda: gated_linear(ag, wg, "relu", act[:, H * D:]), 2 * (B * width + 2 * ff * width + B * ff), 4.0 * B * ff * width)
            xr, yr = mk(B, width, dt=F32), mk(B, width)
            put(f"decode stream_norms ({B})", "decode stream_update", lambda: X.stream_norms(xr, 1e-5, BF, w, w, y=yr, mult=0.5), B * width * 14)
            kc = HybridCache([KvShape(G, D, D)], B, CONTEXT, 64, "cuda", BF)
            for _, kp, vp in kc.kv.values():
                kp.normal_()
                vp.normal_()
            p1, s1 = torch.full((B,), CONTEXT - 1, device="cuda", dtype=torch.int32), torch.arange(B, device="cuda", dtype=torch.int32)
            c1, q1, qkv1 = rotary.angles(p1, freq), mk(B, H, D), mk(B, (H + 2 * G) * D)
            put(f"decode kv_rotate_append ({B})", "decode stream_update",
                lambda: kc.rotate_append(0, qkv1[:, :H * D], qkv1[:, H * D:(H + G) * D], qkv1[:, (H + G) * D:], c1, c1, H, D, s1, p1, 1e-5, False), B * D * (4 * H + 8 * G + 8))
            put(f"attention over pages ({B} x {CONTEXT})", "latent attention", lambda: kc.attention(0, q1, s1, p1, D ** -0.5, CONTEXT, act[:, :H * D], 0, True, c1),
                B * CONTEXT * G * D * 4 + 4 * B * H * D, 4.0 * B * CONTEXT * H * D)
            for mode, name in ((R.BOUNDED, "hgrn2"), (R.ROOT, "gla")):
                args, by, _ = recurrence(B, 1, mode)
                put(f"recurrence, one token, {name} ({B})", "latent attention", lambda: R.advance(*args), by)
    out = {"width": width, "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": src}, "kernels": rows}
    if not alone:
        out["others"] = other.kernel_part(width, iters)["kernels"]
    return out


def run(size="all", part="all", iters=10, alone=False):
    out = {"metric": "nufalorn serving tokens/s beside surelorn and llama at equal size", "dtype": "bf16", "data": "synthetic (random weights and token ids)",
           "l2": "model: weights larger than L2 are streamed every call; kernels: 256 MiB written between calls", "sizes": []}
    for width in SIZES if size == "all" else (int(size),):
        rec = {"width": width}
        if part in ("model", "all"):
            rec["model"] = model_part(width, iters, alone=alone)
        if part in ("kernels", "all"):
            rec["kernels"] = kernel_part(width, max(iters, 10), alone)
        out["sizes"].append(rec)
    return out


def main():
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--size", default="all", choices=["all"] + [str(k) for k in SIZES])
    ap.add_argument("--part", default="all", choices=["model", "kernels", "all"])
    ap.add_argument("--iters", type=int, default=10)
    ap.add_argument("--alone", action="store_true")
    a = ap.parse_args()
    print(json.dumps(run(a.size, a.part, a.iters, a.alone)), flush=True)


if __name__ == "__main__":
    main()
