"""Surelorn beside Llama at equal size (random weights): prompt and decode throughput, and a table of kernels.

    python benchmarks/surelorn.py [--size 2048|4096|all] [--part model|kernels|all] [--iters 20]

``model``: tokens/s of a prompt batch (hidden states and the logits of the last position) and of decoding one token per
sequence at a context of 2048, for Surelorn (bf16) and for the framework's Llama of the same width, heads, feed-forward
size and depth - its bf16 module for prompts and its INT4 engine (INT4 weights and cache, an eighth to a quarter of the bytes) for decoding.
Decode steps of both are CUDA-graph replays.
``kernels``: each kernel of a Surelorn step and the like kernel of a Llama step on the shapes of that size: device time
(median, L2 flushed by a 256 MiB write between calls, graph replay), the time its bytes or FLOPs need at the measured
peaks, and the ratio of the two.
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

# width -> attention and feed-forward sizes; half of the layers are dense, half mixtures
SIZES = {2048: dict(heads=16, dim=128, q_rank=768, kv_rank=512, ff=5632, experts=64, top=6, expert_ff=1408, shared=2816, layers=8, kv_heads=16),
         4096: dict(heads=32, dim=128, q_rank=1536, kv_rank=512, ff=11008, experts=64, top=8, expert_ff=1408, shared=2816, layers=8, kv_heads=32)}
VOCAB, CONTEXT = 32000, 2048
BF = torch.bfloat16


def surelorn_config(width, s, mixture):
    from cogito_b200.models.surelorn import SurelornConfig
    m = {"heads": s["heads"], "dim": s["dim"], "vdim": s["dim"], "q_rank": s["q_rank"], "kv_rank": s["kv_rank"], "scale": s["dim"] ** -0.5}
    dense = {"kind": "dense", "ff": s["ff"]}
    moe = {"kind": "moe", "expert": {"ff": s["expert_ff"]}, "shared": {"ff": s["shared"]},
           "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": 8, "keep": 4}}}
    layers = [{"type": "latent_attention", "mixer": m, "mlp": moe if mixture and i % 2 else dense} for i in range(s["layers"])]
    return SurelornConfig.from_dict({"vocab": VOCAB, "width": width, "embedding": {"scale": width ** 0.5}, "norm": {"eps": 1e-6}, "layers": layers})


def _timed(fn, iters):
    for _ in range(3):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def _graph(fn):
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        fn()
        fn()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        fn()
    return g.replay


def model_part(width, iters=10, prompts=((1, 2048), (4, 2048)), batches=(1, 16, 64), kinds=("dense", "mixture")):
    """Every timed region streams more weights than L2 holds."""
    from cogito_b200.models.llama import Llama, LlamaConfig
    from cogito_b200.models.surelorn import Surelorn, random_tensors
    from cogito_b200.serve.engine import LlamaInt4Engine
    from cogito_b200.serve.stack import StackEngine, TokenBatch
    s = SIZES[width]
    dev = torch.device("cuda")
    out = {"width": width, **{k: s[k] for k in ("heads", "layers", "ff", "kv_rank")}, "context": CONTEXT}
    for kind in kinds:
        cfg = surelorn_config(width, s, kind == "mixture")
        model = Surelorn(cfg, random_tensors(cfg, 0, dev), dev, BF)
        rec = {"params": model.num_params()}
        for B, T in prompts:
            e = StackEngine(model, B, T)
            ids = torch.randint(0, VOCAB, (B, T), device=dev)

            def prompt():
                e.reset()
                pos = torch.arange(T, device=dev, dtype=torch.int32).repeat(B)
                slot = torch.arange(B, device=dev, dtype=torch.int32).repeat_interleave(T)
                from cogito_b200.serve.stack import Segment
                b = TokenBatch(ids.view(-1), pos, slot, [Segment(0, B, T, 0, 0)], B * T, T)
                return model.logits(model.stream(b, e.cache), torch.arange(T - 1, B * T, T, device=dev))
            with torch.no_grad():
                ms = _timed(prompt, iters)
            rec[f"prompt_{B}x{T}"] = {"ms": round(ms, 3), "tok_per_s": round(B * T / ms * 1e3)}
            del e
        for B in batches:
            e = StackEngine(model, B, CONTEXT + 64)
            e.cache.lengths.fill_(CONTEXT)
            e._fresh = False
            tok = torch.randint(0, VOCAB, (B, 1), device=dev)
            ms = _timed(_graph(lambda: e.forward(tok)), iters)
            rec[f"decode_{B}"] = {"ms": round(ms, 3), "tok_per_s": round(B / ms * 1e3)}
            del e
        out[f"surelorn_{kind}"] = rec
        del model
        torch.cuda.empty_cache()
    lc = LlamaConfig(vocab_size=VOCAB, n_layer=s["layers"], d_model=width, n_head=s["heads"], n_kv_head=s["kv_heads"], d_ff=s["ff"], max_seq_len=CONTEXT + 64)
    llama = Llama(lc, device=dev, dtype=BF)
    rec = {"params": llama.num_params()}
    for B, T in prompts:
        ids = torch.randint(0, VOCAB, (B, T), device=dev)
        with torch.no_grad():
            ms = _timed(lambda: llama.lm_head(llama.hidden(ids)[:, -1]), iters)
        rec[f"prompt_{B}x{T}"] = {"ms": round(ms, 3), "tok_per_s": round(B * T / ms * 1e3)}
    for B in batches:
        e = LlamaInt4Engine(llama, B, CONTEXT + 64)
        e.cache.lengths.fill_(CONTEXT)
        e._fresh = False
        tok = torch.randint(0, VOCAB, (B, 1), device=dev)
        with torch.no_grad():
            ms = _timed(_graph(lambda: e.forward(tok)), iters)
        rec[f"decode_int4_{B}"] = {"ms": round(ms, 3), "tok_per_s": round(B / ms * 1e3)}
        del e
    out["llama"] = rec
    del llama
    torch.cuda.empty_cache()
    return out


def kernel_part(width, iters=20):
    from kernels import Timer, peaks
    from cogito_b200.nn.latent_attention import LatentSpec
    from cogito_b200.ops import misc as M
    from cogito_b200.ops import moe as X
    from cogito_b200.ops import stream as R
    from cogito_b200.ops.attention import flash_forward
    from cogito_b200.ops.linear import gated_linear, linear
    from cogito_b200.ops.norm import norm_forward_raw
    from cogito_b200.quant.int4 import Int4Linear
    from cogito_b200.serve.kv_cache import PagedKVCacheInt4, PagedLatentCache
    hbm, tf, src = peaks()
    s, t, rows = SIZES[width], Timer(iters, 3), []
    H, D, R_, q, ff = s["heads"], s["dim"], s["kv_rank"], s["q_rank"], s["ff"]
    mk = lambda *shape, dt=BF: torch.randn(*shape, device="cuda").to(dt)

    def put(name, like, fn, bytes_=0, flops=0, **extra):
        ms = t(fn, graph=True)
        floor = max(bytes_ / hbm / 1e6, flops / tf / 1e9)
        rows.append({"kernel": name, "like": like, "us": round(ms * 1e3, 2), "roofline_us": round(floor * 1e3, 2),
                     "fraction": round(floor / ms, 3), "bound": "hbm" if bytes_ / hbm / 1e6 >= flops / tf / 1e9 else "tensor", **extra})

    def product(name, like, M_, N_, K_, out=BF):
        a, b = mk(M_, K_), mk(N_, K_)
        put(name, like, lambda: linear(a, b, out_dtype=out), 2 * (M_ * K_ + N_ * K_) + (4 if out == torch.float32 else 2) * M_ * N_, 2.0 * M_ * N_ * K_,
            shape=[M_, N_, K_])

    with torch.no_grad():
        T = 4096
        one = torch.zeros(1, device="cuda")
        put("smallest launch (what the method itself costs)", "-", lambda: one.add_(1))
        # ---- prompt: row kernels
        x, y, w = mk(T, width, dt=torch.float32), mk(T, width), torch.ones(width, device="cuda")
        put("stream_update", "norm", lambda: R.stream_update(x, y, w, 1e-6, BF), T * width * (2 + 4 + 4 + 2))
        ids, pos = torch.randint(0, VOCAB, (T,), device="cuda"), torch.arange(T, device="cuda", dtype=torch.int32)
        table, freq = mk(VOCAB, width), R.sinusoid_frequencies(width, device="cuda")
        put("embed_sinusoid", "embedding", lambda: R.embed_sinusoid(ids, pos, table, 2.0, freq), T * width * (2 + 4 + 2))
        ids2 = ids.view(1, T)
        put("llama: embedding", "embedding", lambda: M.embedding(ids2, table, None), T * width * 4)
        xb, yb, wb = mk(T, width), mk(T, width), mk(width)
        put("llama: rms_norm + residual", "norm", lambda: norm_forward_raw(xb, wb, None, 1e-6, True, yb, want_sum=True), T * width * 8)
        cache = PagedLatentCache([R_], 2, T, 64, "cuda", BF)
        slot = torch.zeros(T, device="cuda", dtype=torch.int32)
        wq, wc = torch.ones(q, device="cuda"), torch.ones(R_, device="cuda")
        lat = mk(T, q + R_, dt=torch.float32)
        put("latent_norm_append", "norm", lambda: cache.norm_append(0, lat, wq, wc, 1e-6, slot, pos, True), T * ((q + R_) * 4 + q * 2 + R_ * 4))
        put("latent_gather", "norm", lambda: cache.gather(0, 0, T), T * R_ * 4)
        # ---- prompt: products and attention
        product("gemm dq|dkv (fp32 out)", "gemm", T, q + R_, width, torch.float32)
        product("gemm uq", "gemm", T, H * D, q)
        product("gemm uk|uv", "gemm", T, 2 * H * D, R_)
        product("gemm o", "gemm", T, width, H * D)
        product("gemm gate|up", "gemm", T, 2 * ff, width)
        product("gemm down", "gemm", T, width, ff)
        product("llama: gemm qkv", "gemm", T, 3 * H * D, width)
        kv = mk(2, T // 2, 2, H, D)
        qq = mk(2, T // 2, H, D)
        att = 2 * 2 * 2 * H * D * (T // 2) ** 2 / 2
        put("flash attention (both models)", "flash", lambda: flash_forward(qq, kv[:, :, 0], kv[:, :, 1], causal=True), 0, att)
        gu = mk(T, 2 * ff)
        put("swiglu (both models)", "swiglu", lambda: M.swiglu(gu), T * ff * 6)
        # ---- prompt: mixture
        E, top, F = s["experts"], s["top"], s["expert_ff"]
        h, wr = mk(T, width), mk(E, width)
        put("gemm router", "gemm", lambda: linear(h, wr, out_dtype=torch.float32), 2 * (T * width + E * width) + 4 * T * E, 2.0 * T * E * width, shape=[T, E, width])
        logits, corr = mk(T, E, dt=torch.float32), torch.zeros(E, device="cuda")
        put("moe_route", "sample", lambda: X.route(logits, corr, E, top, 8, 4), T * E * 4 + T * top * 12)
        wgu, wdn = mk(E, 2 * F, width) * width ** -0.5, mk(E, width, F) * F ** -0.5
        for n in (T, 64, 16):
            hn, ln = h[:n].contiguous(), logits[:n].contiguous()
            used = len(set(torch.topk(ln, top)[1].view(-1).tolist())) if n < T else E
            wbytes = used * 3 * F * width * 2
            act = n * top

            def run():
                r = X.route(ln, corr, E, top, count=True)
                return X.expert_outputs(hn, r, wgu, wdn)
            put(f"experts, all steps ({n} tokens)", "gemm" if n == T else "decode gemm", run, wbytes + act * 2 * (2 * width + 5 * F), act * 6.0 * F * width)
        for n in (1, 4):
            hn, ln = h[:n].contiguous(), logits[:n].contiguous()

            def few():
                return X.expert_outputs(hn, X.route(ln, corr, E, top), wgu, wdn)
            put(f"experts, pair by pair ({n} tokens)", "decode gemm", few, len(set(torch.topk(ln, top)[1].view(-1).tolist())) * 3 * F * width * 2)
        rows_y, r = mk(T * top, width), X.route(logits, corr, E, top)
        put("stream_update with expert rows", "norm", lambda: R.stream_update(x, y, w, 1e-6, BF, rows_y, r.row_of, r.weight), T * width * (12 + 2 * top))
        del rows_y, wgu, wdn
        # ---- decode
        for B in (1, 16, 64):
            product(f"decode gemm dq|dkv ({B})", "decode gemm", B, q + R_, width, torch.float32)
            ag, wg = mk(B, width), mk(2 * ff, width)
            put(f"decode gate|up with swiglu ({B})", "decode gemm", lambda: gated_linear(ag, wg), 2 * (B * width + 2 * ff * width + B * ff), 4.0 * B * ff * width)
            product(f"decode gemm down ({B})", "decode gemm", B, width, ff)
            product(f"decode gemm head ({B})", "decode gemm", B, VOCAB, width, torch.float32)
            qh, wk, qa = mk(B, H, D), mk(H, D, R_), mk(B, H, R_)
            put(f"decode product W_uk^T q ({B})", "decode gemm", lambda: linear(qh.transpose(0, 1), wk, w_mn=True, out=qa.transpose(0, 1)), 2 * H * D * R_ + 2 * B * H * (D + R_))
            lc = PagedLatentCache([R_], B, CONTEXT, 64, "cuda", BF)
            lc.pages[0].normal_()
            p1 = torch.full((B,), CONTEXT - 1, device="cuda", dtype=torch.int32)
            s1 = torch.arange(B, device="cuda", dtype=torch.int32)
            put(f"latent attention ({B} x {CONTEXT})", "decode attention", lambda: lc.attention(0, qa, s1, p1, 0.1, CONTEXT),
                B * CONTEXT * R_ * 2 + 4 * B * H * R_, 4.0 * B * CONTEXT * H * R_)
            xr, yr = mk(B, width, dt=torch.float32), mk(B, width)
            put(f"decode stream_update ({B})", "decode norm", lambda: R.stream_update(xr, yr, w, 1e-6, BF), B * width * 12)
            xb1, yb1 = mk(B, width), mk(B, width)
            put(f"llama: decode rms_norm + residual ({B})", "decode norm", lambda: norm_forward_raw(xb1, wb, None, 1e-6, True, yb1, want_sum=True), B * width * 8)
            for name, n_, k_ in (("qkv", 3 * H * D, width), ("gate|up", 2 * ff, width), ("down", width, ff), ("head", VOCAB, width)):
                lin = Int4Linear(torch.randn(n_, k_, device="cuda") * 0.02, None, 128)
                xx = mk(B, k_)
                put(f"llama: int4 gemm {name} ({B})", "decode gemm", lambda: lin(xx), n_ * k_ * (0.5 + 4 / 128) + 2 * B * (n_ + k_), 2.0 * B * n_ * k_)
            kc = PagedKVCacheInt4(1, B, CONTEXT, s["kv_heads"], D, 32, 64, "cuda")
            kc.lengths.fill_(CONTEXT - 1)
            q1 = mk(B, 1, H, D)
            put(f"llama: int4 kv attention ({B} x {CONTEXT})", "decode attention", lambda: kc.attention(0, q1), B * CONTEXT * s["kv_heads"] * D * 2 * (0.5 + 4 / 32),
                4.0 * B * CONTEXT * H * D)
    return {"width": width, "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": src}, "kernels": rows}


def run(size="all", part="all", iters=10):
    out = {"metric": "surelorn serving tokens/s beside llama at equal size", "dtype": "bf16", "data": "synthetic (random weights and token ids)",
           "l2": "model: weights larger than L2 are streamed every call; kernels: 256 MiB written between calls", "sizes": []}
    for width in SIZES if size == "all" else (int(size),):
        rec = {"width": width}
        if part in ("model", "all"):
            rec["model"] = model_part(width, iters)
        if part in ("kernels", "all"):
            rec["kernels"] = kernel_part(width, max(iters, 10))
        out["sizes"].append(rec)
    return out


def main():
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--size", default="all", choices=["all"] + [str(k) for k in SIZES])
    ap.add_argument("--part", default="all", choices=["model", "kernels", "all"])
    ap.add_argument("--iters", type=int, default=10)
    a = ap.parse_args()
    print(json.dumps(run(a.size, a.part, a.iters)), flush=True)


if __name__ == "__main__":
    main()
