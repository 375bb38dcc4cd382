"""Surelorn on a B200: each kernel against a slow restatement, and the engine (bf16 and fp32) against
plain_surelorn.py: prompts, portions, decoding, batches, reused pages, key borders, sampling and graphs."""
import pytest
import torch

import plain_surelorn as plain
import surelorn_cases as S
from cogito_b200.ops import _lib
from cogito_b200.ops import moe as X
from cogito_b200.ops import stream as R
from cogito_b200.ops.gemm import gemm
from cogito_b200.serve.kv_cache import PagedLatentCache

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
DEV = "cuda"


@pytest.fixture(autouse=True)
def _device_status():
    yield
    if torch.cuda.is_available():
        _lib.assert_device_ok()


def rand(*shape, seed=0, dtype=F32, scale=1.0):
    g = torch.Generator().manual_seed(seed + sum(shape))
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


# ------------------------------------------------------------------ kernels
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width", [64, 130, 7])
def test_embedding_with_sinusoid(dtype, width):
    table = rand(50, width, dtype=dtype)
    ids = torch.randint(0, 50, (9,))
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 4097, 30000, 131071], dtype=torch.int32)
    freq = R.sinusoid_frequencies(width)
    x, h = R.embed_sinusoid(ids.to(DEV), pos.to(DEV), table.to(DEV), 1.75, freq.to(DEV))
    want = table[ids].double() * 1.75 + plain.sinusoid(pos.tolist(), width)
    assert torch.allclose(x.cpu().double(), want, atol=2e-6) and torch.equal(h.cpu(), x.cpu().to(dtype))


@pytest.mark.parametrize("D", [96, 352, 4096, 6144, 130, 33])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_stream_update_and_final_norm(D, dtype):
    N, P, top = 11, 20, 3
    x0, w = rand(N, D, seed=1, scale=4.0), torch.rand(D) + 0.5
    for y_dt, p_dt, with_y, with_p in [(dtype, dtype, True, False), (dtype, F32, False, True), (F32, dtype, True, True), (F32, F32, True, True)]:
        if dtype == F32 and BF in (y_dt, p_dt):
            continue
        y = rand(N, D, seed=2, dtype=y_dt) if with_y else None
        pairs = rand(P, D, seed=3, dtype=p_dt) if with_p else None
        row_of = torch.randint(-1, P, (N, top), generator=torch.Generator().manual_seed(4)).to(torch.int32)
        weight = torch.rand(N, top)
        v = y.double() if with_y else torch.zeros(N, D, dtype=torch.float64)
        if with_p:
            for t in range(N):
                for k in range(top):
                    r = int(row_of[t, k])
                    v[t] += weight[t, k].double() * (pairs[r].double() if r >= 0 else x0[t].double())
        want = x0.double() + plain.rms(v, w.double(), 1e-4)
        x = x0.to(DEV)
        kw = dict(pairs=pairs.to(DEV), row_of=row_of.to(DEV), weight=weight.to(DEV)) if with_p else {}
        h = R.stream_update(x, y.to(DEV) if with_y else None, w.to(DEV), 1e-4, dtype, **kw)
        assert torch.allclose(x.cpu().double(), want, atol=5e-5, rtol=1e-5)
        assert h.dtype == dtype and torch.equal(h.cpu(), x.cpu().to(dtype))
    rows = torch.tensor([10, 0, 3])
    got = R.rms_rows(x, w.to(DEV), 1e-4, F32, rows.to(DEV))
    assert torch.allclose(got.cpu().double(), plain.rms(x.cpu().double(), w.double(), 1e-4)[rows], atol=2e-5)


@pytest.mark.parametrize("b_mn", [False, True])
def test_fp32_product_is_not_a_reduced_precision_one(b_mn):
    for M, N, K, B in [(70, 130, 33, 1), (1, 5, 600, 3), (129, 64, 16, 2)]:
        a, b = rand(B, M, K, seed=5), rand(B, K, N, seed=6) if b_mn else rand(B, N, K, seed=6)
        got = gemm(a.to(DEV), b.to(DEV), b_mn=b_mn)
        want = a.double() @ (b.double() if b_mn else b.double().transpose(1, 2))
        assert float((got.cpu().double() - want).abs().max()) < 2e-5 * K ** 0.5
    # strided batches: heads interleaved in the rows
    a, w = rand(6, 4 * 10, seed=7).to(DEV), rand(4, 10, 12, seed=8).to(DEV)
    out = torch.empty(6, 4, 12, device=DEV)
    gemm(a.view(6, 4, 10).transpose(0, 1), w, b_mn=True, out=out.transpose(0, 1))
    assert torch.allclose(out.cpu().double(), torch.einsum("nhk,hkr->nhr", a.view(6, 4, 10).cpu().double(), w.cpu().double()), atol=1e-4)


@pytest.mark.parametrize("M", [1, 2, 3, 5, 8, 9])
@pytest.mark.parametrize("N,K", [(3, 8), (100, 264), (2500, 520), (12001, 64), (40, 4104)])
def test_products_with_few_rows(M, N, K):
    from cogito_b200.ops.linear import gated_linear, linear
    a, w = rand(M, K, seed=1, dtype=BF), rand(N, K, seed=2, dtype=BF, scale=K ** -0.5)
    want = a.double() @ w.double().T
    for dt, tol in ((F32, 2e-5), (BF, 1e-2)):
        got = linear(a.to(DEV), w.to(DEV), out_dtype=dt)
        assert got.dtype == dt and float((got.cpu().double() - want).abs().max()) < tol * max(1.0, float(want.abs().max()))
    w2 = rand(2 * N, K, seed=3, dtype=BF, scale=K ** -0.5)
    want = plain.silu(a.double() @ w2[:N].double().T) * (a.double() @ w2[N:].double().T)
    got = gated_linear(a.to(DEV), w2.to(DEV))
    assert float((got.cpu().double() - want).abs().max()) < 2e-2 * max(1.0, float(want.abs().max()))
    # heads interleaved in the rows, both storage orders
    H, D, R = 3, 40, 136
    x, wk, wv = rand(M, H * D, seed=4, dtype=BF), rand(H, D, R, seed=5, dtype=BF), rand(H, D, R, seed=6, dtype=BF)
    xh, up = x.to(DEV).view(M, H, D).transpose(0, 1), torch.empty(M, H, R, dtype=BF, device=DEV)
    linear(xh, wk.to(DEV), w_mn=True, out=up.transpose(0, 1))
    want = torch.einsum("mhd,hdr->mhr", x.view(M, H, D).double(), wk.double())
    assert float((up.cpu().double() - want).abs().max()) < 1e-2 * float(want.abs().max())
    down = torch.empty(M, H * D, dtype=BF, device=DEV)
    linear(up.transpose(0, 1), wv.to(DEV), out=down.view(M, H, D).transpose(0, 1))
    want = torch.einsum("mhr,hdr->mhd", up.cpu().double(), wv.double()).reshape(M, H * D)
    assert float((down.cpu().double() - want).abs().max()) < 1e-2 * float(want.abs().max())


def _latents(R, dtype, lengths, page_size=64, seed=0, extra_pages=3):
    """A cache whose sequences own shuffled pages, filled with the given numbers of random latents."""
    g = torch.Generator().manual_seed(seed)
    pages = sum((n + page_size - 1) // page_size for n in lengths) + extra_pages
    c = PagedLatentCache([R], len(lengths), max(lengths), page_size, DEV, dtype, n_pages=pages)
    perm = torch.randperm(pages, generator=g).tolist()
    c._free_pages = perm
    data = []
    for n in lengths:
        s = c.open()
        c.reserve(s, n)
        lat = torch.randn(n, R, generator=g).to(dtype)
        page = c.page_table[s, torch.arange(n, device=DEV) // page_size].long()
        c.pages[0][page, torch.arange(n, device=DEV) % page_size] = lat.to(DEV)
        data.append((s, lat.double()))
    return c, data


def _attend(q, lat, pos, scale):
    s = q.double() @ lat[:pos + 1].T * scale
    return torch.softmax(s, -1) @ lat[:pos + 1]


SHAPES = [(128, 6), (128, 17), (96, 3), (64, 33), (512, 16), (512, 40), (256, 64), (72, 5), (384, 8), (36, 6), (40, 2), (33, 3), (1024, 2)]


@pytest.mark.parametrize("rank,heads", SHAPES)
@pytest.mark.parametrize("dtype", [BF, F32])
def test_latent_attention_over_pages(rank, heads, dtype):
    """Random soft scores, unequal sequences, positions on both sides of every kind of border."""
    lengths = [1, 2, 63, 64, 65, 127, 128, 129, 700, 1500]
    c, data = _latents(rank, dtype, lengths, seed=rank)
    slot, pos, want = [], [], []
    q = rand(len(lengths) + 4, heads, rank, seed=9, dtype=dtype)
    scale = 1.5 * rank ** -0.5
    places = [(i, n - 1) for i, n in enumerate(lengths)] + [(8, 0), (8, 256), (9, 767), (9, 768)]
    for i, (k, p) in enumerate(places):
        slot.append(data[k][0])
        pos.append(p)
        want.append(_attend(q[i], data[k][1], p, scale))
    want = torch.stack(want)
    s, p = torch.tensor(slot, dtype=torch.int32, device=DEV), torch.tensor(pos, dtype=torch.int32, device=DEV)
    tol = 1e-5 if dtype == F32 else 1.2e-2
    for max_len in (1500, 64):                             # many key ranges, one key range
        got = c.attention(0, q.to(DEV), s, p, scale, max_len).cpu().double()
        assert float((got - want).abs().max()) < tol * float(want.abs().max()), max_len
    if dtype == BF:
        got = c.attention(0, q.to(DEV), s, p, scale, 1500, force_simt=True).cpu().double()
        assert float((got - want).abs().max()) < tol * float(want.abs().max())


@pytest.mark.parametrize("rank,heads", [(128, 6), (512, 20), (256, 40), (36, 3)])
def test_one_standing_out_key_is_found_anywhere_and_the_next_one_is_not_seen(rank, heads):
    n = 1100
    for dtype in (BF, F32):
        c, [(slot, lat)] = _latents(rank, dtype, [n], seed=3)
        pos, q, want = [], [], []
        for at in (0, 1, 62, 63, 64, 65, 127, 128, 255, 256, 511, 512, 1023, 1024, n - 2, n - 1):
            for query in sorted({at, min(at + 1, n - 1), n - 1, max(at - 1, 0)}):
                pos.append(query)
                q.append((lat[at] / lat[at].norm() * 3.0).to(dtype).expand(heads, rank))
                want.append(_attend(q[-1], lat, query, 4.0))
        q, want = torch.stack(q), torch.stack(want)
        N = len(pos)
        got = c.attention(0, q.to(DEV).contiguous(), torch.full((N,), slot, dtype=torch.int32, device=DEV),
                          torch.tensor(pos, dtype=torch.int32, device=DEV), 4.0, n).cpu().double()
        assert float((got - want).abs().max()) < (1e-4 if dtype == F32 else 2e-2) * float(want.abs().max())


def test_growing_scores_rescale_the_accumulator():
    """Keys whose scores climb by far more than 2^8 from block to block, and fall again."""
    rank, heads, n = 128, 5, 900
    c, [(slot, _)] = _latents(rank, BF, [n], seed=1)
    lat = rand(n, rank, seed=2, scale=0.05)
    lat[:, 0] = torch.sin(torch.arange(n) / 140.0) * 3 + torch.arange(n) / 300.0
    lat = lat.to(BF)
    page = c.page_table[slot, torch.arange(n, device=DEV) // 64].long()
    c.pages[0][page, torch.arange(n, device=DEV) % 64] = lat.to(DEV)
    q = rand(8, heads, rank, seed=4, scale=0.3)
    q[..., 0] = 20.0
    q = q.to(BF)
    pos = [100, 128, 300, 420, 600, 760, 850, n - 1]
    want = torch.stack([_attend(q[i], lat.double(), p, 0.5) for i, p in enumerate(pos)])
    for max_len in (n, 64):
        got = c.attention(0, q.to(DEV), torch.full((8,), slot, dtype=torch.int32, device=DEV), torch.tensor(pos, dtype=torch.int32, device=DEV), 0.5, max_len)
        assert float((got.cpu().double() - want).abs().max()) < 1e-2 * float(want.abs().max())


@pytest.mark.parametrize("in_dtype,dtype", [(F32, BF), (BF, BF), (F32, F32)])
def test_norm_append_and_gather(in_dtype, dtype):
    qr, R, N = 40, 72, 150
    c = PagedLatentCache([R], 2, 200, 64, DEV, dtype, n_pages=6)
    c._free_pages = [3, 0, 5, 2, 4, 1]
    a = c.open()
    c.reserve(a, 170)
    lat, wq, wc = rand(N, qr + R, seed=1, dtype=in_dtype), torch.rand(qr), torch.rand(R)
    pos = torch.arange(20, 170, dtype=torch.int32)
    cq, cc = c.norm_append(0, lat.to(DEV), wq.to(DEV), wc.to(DEV), 1e-5, torch.full((N,), a, dtype=torch.int32, device=DEV), pos.to(DEV), True)
    wantc, wantq = plain.rms(lat[:, qr:].double(), wc.double(), 1e-5), plain.rms(lat[:, :qr].double(), wq.double(), 1e-5)
    tol = 1e-5 if dtype == F32 else 1e-2
    assert torch.allclose(cq.cpu().double(), wantq, atol=tol) and torch.allclose(cc.cpu().double(), wantc, atol=tol)
    got = c.gather(0, a, 170)
    assert torch.equal(got[20:], cc) and float(got[:20].abs().max()) == 0.0


@pytest.mark.parametrize("experts,identity,top,groups,keep", [(6, 2, 3, 4, 2), (5, 0, 2, 1, 1), (120, 8, 8, 8, 3), (250, 6, 16, 64, 20), (1, 0, 1, 1, 1),
                                                              (4, 4, 1, 2, 1), (1000, 24, 5, 128, 2)])
def test_routing(experts, identity, top, groups, keep):
    O, N = experts + identity, 70
    logits, corr = rand(N, O, seed=1, scale=2.0), rand(O, seed=2, scale=0.3) - 0.2
    r = X.route(logits.to(DEV), corr.to(DEV), experts, top, groups, keep, count=True)
    hist = torch.zeros(experts, dtype=torch.int64)
    for t in range(N):
        want = plain.choose(logits[t].double(), corr.double(), {"groups": {"count": groups, "keep": keep}, "top": top})
        assert r.idx[t].tolist() == [i for i, _ in want]
        assert torch.allclose(r.weight[t].cpu().double(), torch.stack([v for _, v in want]), atol=1e-6)
        assert [v >= 0 for v in r.row_of[t].tolist()] == [i < experts for i, _ in want]
        for i, _ in want:
            if i < experts:
                hist[i] += 1
    assert torch.equal(r.counts.cpu().long(), hist)
    r.counts.zero_()


@pytest.mark.parametrize("N,D,F,E,identity,top", [(1, 64, 32, 4, 1, 2), (7, 96, 40, 6, 2, 3), (300, 128, 64, 5, 3, 2), (40, 256, 160, 70, 2, 6), (513, 64, 96, 3, 0, 1),
                                                  (50, 130, 30, 5, 1, 2), (2000, 352, 96, 10, 2, 3)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_expert_outputs(N, D, F, E, identity, top, dtype):
    h, gu, dn = rand(N, D, seed=1, dtype=dtype), rand(E, 2 * F, D, seed=2, dtype=dtype, scale=D ** -0.5), rand(E, D, F, seed=3, dtype=dtype, scale=F ** -0.5)
    logits = rand(N, E + identity, seed=4)
    logits[:, 0] += 1.5                                    # unequal loads
    hd, gud, dnd = h.to(DEV), gu.to(DEV), dn.to(DEV)
    for grouped in (False, True):
        if grouped and not X.grouped_ok(hd, gud, dnd):
            continue
        for _ in range(2):                                 # the counters are clean again after a call
            r = X.route(logits.to(DEV), torch.zeros(E + identity, device=DEV), E, top, count=grouped)
            rows = X.expert_outputs(hd, r, gud, dnd).cpu().double()
        idx, row_of = r.idx.cpu(), r.row_of.cpu()
        worst = scale = 0.0
        for t in range(0, N, max(1, N // 60)):
            for k in range(top):
                e = int(idx[t, k])
                assert (int(row_of[t, k]) >= 0) == (e < E)
                if e < E:
                    want = plain.gated(h[t:t + 1].double(), gu[e, :F].double(), gu[e, F:].double(), dn[e].double())[0]
                    worst = max(worst, float((rows[int(row_of[t, k])] - want).abs().max()))
                    scale = max(scale, float(want.abs().max()))
        assert worst < (1e-5 if dtype == F32 else 2e-2) * scale
        if grouped:
            assert int(r.counts.abs().sum()) == 0 and len(set(row_of[row_of >= 0].tolist())) == int((row_of >= 0).sum())


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", ["mixed", "odd", "wide", "long_heads"])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_prompts_portions_and_decoding_match_the_restatement(name, dtype):
    d, cfg, t = S.build(name)
    n = 150
    toks = S.tokens(n, cfg.vocab_size, 1)
    want = S.expect(d, t, toks)
    e = S.engine(cfg, t, DEV, dtype)
    for cuts in ([(0, n)], [(i, 1) for i in range(n)], S.portions(n, [33, 2, 64, 5]), S.portions(n, [2]), [(0, 60), (60, 32)] + [(i, 1) for i in range(92, n)]):
        S.assert_close(S.feed(e, toks, cuts), want, dtype, (name, cuts[:3]))
    eager = S.engine(cfg, t, DEV, dtype, use_graph=False)
    S.assert_close(S.feed(eager, toks, [(i, 1) for i in range(n)]), want, dtype, "without graphs")


def test_every_layer_of_the_stream_matches():
    for name in ("mixed", "wide"):
        d, cfg, t = S.build(name, 3)
        toks = S.tokens(40, cfg.vocab_size, 4)
        want, got = [], []
        plain.forward(d, t, toks, keep=want)
        e = S.engine(cfg, t, DEV, F32)
        e.step([(e.open(), toks, [])], keep=got)
        for i, (a, b) in enumerate(zip(got, want)):
            assert float((a.cpu().double() - b).abs().max()) < 3e-4, (name, i)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_batches_of_unequal_sequences_and_pages_used_again(dtype):
    d, cfg, t = S.build("mixed", 5)
    seqs = [S.tokens(n, cfg.vocab_size, 10 + n) for n in (190, 3, 137, 18)]
    want = [S.expect(d, t, s) for s in seqs]
    e = S.engine(cfg, t, DEV, dtype, pool=448)
    for _ in range(3):
        slots = [e.open() for _ in seqs]
        at, got = [0] * 4, [[] for _ in seqs]
        for row in [(140, 2, 0, 17), (1, 1, 65, 1), (40, 0, 2, 0), (1, 0, 1, 0), (8, 0, 69, 0)]:
            part = [(i, n) for i, n in enumerate(row) if n]
            out = e.step([(slots[i], seqs[i][at[i]:at[i] + n], list(range(n))) for i, n in part]).double().cpu()
            for i, n in part:
                got[i].append(out[:n])
                out = out[n:]
                at[i] += n
        for i in range(4):
            S.assert_close(torch.cat(got[i]), want[i], dtype, i)
            e.close(slots[i])


def test_long_decoding_and_far_keys_in_fp32():
    """700 tokens, most of them decoded one by one: in fp32 a single lost or extra key among hundreds is visible."""
    d = S.config(48, 60, [S.layer(S.mixer(2, 16, 16, 24, 40, 0.6), S.dense(32)), S.layer(S.mixer(2, 16, 16, 24, 40, 0.6), S.dense(32), 0)])
    cfg = S.SurelornConfig.from_dict(d)
    t = S.random_tensors(cfg, 2)
    toks = S.tokens(700, 60, 3)
    want = S.expect(d, t, toks)
    e = S.engine(cfg, t, DEV, F32)
    S.assert_close(S.feed(e, toks, [(0, 90)] + [(i, 1) for i in range(90, 700)]), want, F32)
    b = S.engine(cfg, t, DEV, BF)
    S.assert_close(S.feed(b, toks, [(0, 90)] + [(i, 1) for i in range(90, 700)]), want, BF)
    S.assert_close(S.feed(b, toks, S.portions(700, [129, 64, 2])), want, BF)


def test_greedy_generation_through_the_scheduler_and_the_command_line(tmp_path):
    import json

    from cogito_b200.cli import main
    from cogito_b200.models.surelorn import save_folder
    from cogito_b200.serve.scheduler import Scheduler
    d, cfg, t = S.build("mixed", 7)
    prompts = [S.tokens(n, cfg.vocab_size, n) for n in (5, 70, 1, 44, 12)]
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(6):
            seq.append(int(S.expect(d, t, seq)[-1].argmax()))
        want.append(seq[len(p):])
    e = S.engine(cfg, t, DEV, F32, slots=3, pool=320)
    s = Scheduler(e, step_tokens=48)
    reqs = [s.add(p, 6) for p in prompts]
    s.run()
    assert [r.tokens for r in reqs] == want
    assert e.free_slots() == 3 and e.cache.free_pages() == e.cache.n_pages - 1
    save_folder(str(tmp_path / "m"), cfg, t)
    (tmp_path / "p.json").write_text(json.dumps(prompts))
    main(["generate", f"model.path={tmp_path}/m", "generate.dtype=float32", f"generate.prompts={tmp_path}/p.json", "generate.new_tokens=6",
          f"generate.out={tmp_path}/o.json"])
    assert json.loads((tmp_path / "o.json").read_text()) == [p + w for p, w in zip(prompts, want)]


def test_speculative_decoding_accepts_its_own_drafts():
    from cogito_b200.models.surelorn import Surelorn
    from cogito_b200.serve.engine import SpeculativeDecoder
    from cogito_b200.serve.stack import StackEngine
    d, cfg, t = S.build("mixed", 7)
    prompts = torch.tensor([S.tokens(40, cfg.vocab_size, 1), S.tokens(40, cfg.vocab_size, 2)])
    m = Surelorn(cfg, t, DEV, F32)
    dec = SpeculativeDecoder(StackEngine(m, 2, 256), StackEngine(m, 2, 256), gamma=3, temperature=0.0)
    seqs, stats = dec.generate(prompts.to(DEV), 12)
    assert stats.acceptance_rate == 1.0
    for b in range(2):
        seq = prompts[b].tolist()
        for _ in range(6):
            seq.append(int(S.expect(d, t, seq)[-1].argmax()))
        assert seqs[b][40:46] == seq[40:]
    dec.close()


def test_trace_runner_program(tmp_path):
    import json
    import subprocess
    import sys
    from pathlib import Path

    import numpy as np

    from cogito_b200.models.surelorn import save_folder
    d, cfg, t = S.build("odd", 2)
    save_folder(str(tmp_path / "m"), cfg, t)
    toks = S.tokens(40, cfg.vocab_size, 1)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:38], "want": [0, 37]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[38:39], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[39:], "want": [0]}], "end": ["a"]}]
    root = Path(__file__).resolve().parent.parent
    r = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "64"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=200)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = S.expect(d, t, toks)
    got = torch.from_numpy(np.concatenate([np.fromfile(tmp_path / f"{i}.f32", dtype="<f4") for i in (0, 2)]).reshape(3, -1)).double()
    S.assert_close(got, want[[0, 37, 39]], F32)
