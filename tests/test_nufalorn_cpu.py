"""Nufalorn on the host path: mechanisms, configuration and files, cache and slots, portions and batches, scheduler,
speculative decoding, command line, trace replay - against the slow restatement in plain_nufalorn.py."""
import io
import json
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import nufalorn_cases as S
import plain_nufalorn as plain
from cogito_b200.models import registry
from cogito_b200.models.nufalorn import Nufalorn, NufalornConfig, random_tensors
from cogito_b200.ops import misc as M
from cogito_b200.ops import recurrence as R
from cogito_b200.ops import rotary
from cogito_b200.ops import stream as X
from cogito_b200.ops.attention import flash_forward
from cogito_b200.serve import trace
from cogito_b200.serve.engine import SpeculativeDecoder
from cogito_b200.serve.hybrid_cache import HybridCache, KvShape, StateShape
from cogito_b200.serve.scheduler import Scheduler, generate
from cogito_b200.serve.stack import StackEngine

F32, F64 = torch.float32, torch.float64


# ------------------------------------------------------------------ the restatement itself
def test_plain_rotation_depends_on_the_distance_alone_and_leaves_the_rest():
    torch.manual_seed(0)
    q, k = torch.randn(10, dtype=F64), torch.randn(10, dtype=F64)
    a = plain.turn(q, 9, 100.0, 6) @ plain.turn(k, 4, 100.0, 6)
    b = plain.turn(q, 25, 100.0, 6) @ plain.turn(k, 20, 100.0, 6)
    assert torch.allclose(a, b) and torch.equal(plain.turn(q, 9, 100.0, 6)[6:], q[6:])
    assert torch.allclose(plain.turn(plain.turn(q, 7, 50.0, 10), 7, 50.0, 10, -1), q)
    one = plain.turn(torch.tensor([1.0, 0, 0, 1], dtype=F64), 1, 100.0, 4)          # angles 1 and 1 / 10
    assert torch.allclose(one, torch.tensor([math.cos(1), math.sin(1), -math.sin(0.1), math.cos(0.1)], dtype=F64))


def test_plain_weights_leave_a_share_to_the_sink_and_blocks_start_at_their_first_position():
    w = plain.sink_weights(torch.tensor([0.0, math.log(2.0)], dtype=F64))
    assert torch.allclose(w, torch.tensor([0.25, 0.5], dtype=F64))
    assert float(plain.sink_weights(torch.tensor([-200.0], dtype=F64))) < 1e-80 and abs(float(plain.sink_weights(torch.tensor([900.0], dtype=F64))) - 1) < 1e-12
    assert [list(plain.visible(i, 3)) for i in range(5)] == [[0], [0, 1], [0, 1, 2], [3], [3, 4]]


def test_plain_recurrence_is_a_decayed_sum():
    torch.manual_seed(1)
    q, k, v, a = torch.randn(6, 2, 3), torch.randn(6, 2, 3), torch.randn(6, 2, 4), torch.rand(6, 2, 3)
    o = plain.recurrence(q, k, v, a)
    want = sum((q[5] * k[s] * a[s + 1:6].prod(0)).sum(-1, keepdim=True) * v[s] for s in range(6))
    assert torch.allclose(o[5], want, atol=1e-5)


# ------------------------------------------------------------------ mechanisms, host form
def test_angles_and_turning():
    pos = torch.tensor([0, 1, 77, 100000], dtype=torch.int32)
    for base, dims in ((10000.0, 8), (3.0, 2), (1e6, 6)):
        cs = rotary.angles(pos, rotary.frequencies(base, dims))
        x = torch.randn(4, 3, dims + 3)
        want = torch.stack([plain.turn(x[i].double(), int(p), base, dims) for i, p in enumerate(pos)])
        assert torch.allclose(rotary.turn(x, cs).double(), want, atol=1e-6)


def test_stream_norms_and_softcap_and_gate():
    torch.manual_seed(0)
    table, ids = torch.randn(9, 7), torch.tensor([3, 8, 0])
    x, w1, w2 = torch.empty(3, 7), torch.rand(7), torch.rand(7)
    h1, h2 = X.stream_norms(x, 1e-3, F32, w1, w2, ids=ids, table=table)
    assert torch.equal(x, table[ids]) and torch.allclose(h2.double(), plain.rms(x.double(), 1e-3) * w2, atol=1e-6)
    before, y = x.clone(), torch.randn(3, 7)
    h1, none = X.stream_norms(x, 1e-3, F32, w1, y=y, mult=0.3)
    assert none is None and torch.allclose(x, before + 0.3 * y) and torch.allclose(h1.double(), plain.rms(x.double(), 1e-3) * w1, atol=1e-6)
    v = torch.tensor([-1e4, -3.0, 0.0, 0.5, 80.0])
    assert torch.allclose(X.softcap(v.clone(), 5.0), 5.0 * torch.tanh(v / 5.0))
    gu = torch.randn(4, 10)
    assert torch.allclose(M.gated(gu, "relu"), torch.clamp(gu[:, :5], min=0) * gu[:, 5:])


@pytest.mark.parametrize("block,sink", [(5, True), (0, True), (1, False), (16, True)])
def test_prompt_attention_with_blocks_sink_and_turned_results(block, sink):
    torch.manual_seed(2)
    T, begin, H, G, d, n = 9, 16, 4, 2, 8, 6
    q, k, v = torch.randn(1, T, H, d), torch.randn(1, T + begin, G, d), torch.randn(1, T + begin, G, d)
    freq = rotary.frequencies(50.0, n)
    turn = rotary.angles(torch.arange(begin, begin + T, dtype=torch.int32), freq)
    out = torch.empty(1, T, H, n)
    flash_forward(q, k, v, causal=True, scale=0.4, out=out, block=block, sink=sink, turn=turn[None])
    for i in range(T):
        p = begin + i
        see = plain.visible(p, block or 10**6)
        for h in range(H):
            s = k[0, see.start:p + 1, h // 2].double() @ q[0, i, h].double() * 0.4
            w = plain.sink_weights(s) if sink else torch.softmax(s, -1)
            want = plain.turn((w @ v[0, see.start:p + 1, h // 2].double())[:n], p, 50.0, n, -1)
            assert torch.allclose(out[0, i, h].double(), want, atol=1e-5)


def _operands(N, H, D, V, mode, seed, gate):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    return R.Operands(r(N, H * D), r(N, H * D) if mode == R.ROOT else None, r(N, H * V), r(N, H * V) if gate else None, 2 * r(N, H * D), r(H * D),
                      0.9 * torch.rand(H * D, generator=g) if mode == R.BOUNDED else None, 1 + 0.2 * r(V))


def plain_advance(rule, x, rows):
    """The rows of one sequence, from position 0."""
    T, H, D, V = len(rows), rule.heads, rule.dim, rule.vdim
    z = (x.z[rows] + x.bias).double()
    if rule.mode == R.ROOT:
        a, k = plain.sigmoid(z) ** (1 / rule.tau), x.k[rows].double()
    else:
        a = x.low.double() + (1 - x.low.double()) * plain.sigmoid(z)
        k = 1 - a
    q = x.q[rows].double()
    q = (plain.silu(q) if rule.q_silu else q) * rule.q_scale
    o = plain.recurrence(q.view(T, H, D), k.view(T, H, D), x.v[rows].double().view(T, H, V), a.view(T, H, D))
    o = (plain.rms(o, rule.eps) * x.w.double()).reshape(T, -1)
    return o if x.gate is None else o * plain.silu(x.gate[rows].double())


@pytest.mark.parametrize("mode", [R.BOUNDED, R.ROOT])
def test_recurrence_over_runs_slots_and_histories(mode):
    H, D, V = 2, 3, 5
    rule = R.StateRule(H, D, V, mode, 1e-4, q_silu=mode == R.BOUNDED, q_scale=0.7, tau=3.0)
    x = _operands(20, H, D, V, mode, 1, gate=mode == R.ROOT)
    want = torch.cat([plain_advance(rule, x, list(range(0, 12))), plain_advance(rule, x, list(range(12, 20)))])
    for history in (1, 4):
        state = torch.full((3, history, H, D, V), 1e30)            # what a slot held before does not matter
        out, done = torch.zeros(20, H * V + 3), [0, 0]
        for parts in ([(0, 5), (12, 2)], [(5, 1)], [(6, 6), (14, 6)]):
            rows = [t for lo, n in parts for t in range(lo, lo + n)]
            sub = R.Operands(*[None if t is None else t[rows] for t in (x.q, x.k, x.v, x.gate, x.z)], x.bias, x.low, x.w)
            pos = torch.tensor([t if t < 12 else t - 12 for t in rows], dtype=torch.int32)
            slot = torch.tensor([2 if t < 12 else 0 for t in rows], dtype=torch.int32)
            first = [rows.index(lo) for lo, _ in parts]
            runs = torch.tensor([[f, n] for f, (_, n) in zip(first, parts)], dtype=torch.int32)
            part = torch.zeros(len(rows), H * V)
            R.advance(rule, sub, state, SimpleNamespace(slot=slot, pos=pos, runs=runs, prompts=[]), part)
            out[rows, :H * V] = part
        assert torch.allclose(out[:, :H * V].double(), want, atol=1e-5)


def test_stretches_cover_every_run_in_whole_chunks():
    for counts in ([64], [8192], [1, 63, 64, 65, 4096], [300] * 200, [100000, 32]):
        for heads in (1, 4, 16, 200):
            rows = [sum(counts[:i]) for i in range(len(counts))]
            items, run_items, cut = R.stretches(counts, heads, rows)
            assert cut == (len(items) > len(counts)) and sum(n for _, n in run_items) == len(items)
            for r, (first, n) in enumerate(run_items):
                mine = items[first:first + n]
                assert [m[2] for m in mine] == [r] * n and [m[3] for m in mine] == [0] * (n - 1) + [1]
                assert sum(m[1] for m in mine) == counts[r] and all(m[1] % R.CHUNK == 0 for m in mine[:-1])
                assert [m[0] for m in mine] == [rows[r] + sum(k[1] for k in mine[:i]) for i in range(n)]


def test_hybrid_cache_keeps_turned_keys_and_values_in_pages():
    torch.manual_seed(3)
    c = HybridCache([KvShape(2, 10, 6), StateShape(1, 4, 4), 0], 3, 20, page_size=4, dtype=F32, n_pages=6)
    assert c.kv[2][1] is c.kv[0][1] and c.history == 1 and list(c.states) == [1]
    a = c.open()
    c.reserve(a, 9)
    pos, slot = torch.arange(9, dtype=torch.int32), torch.full((9,), a, dtype=torch.int32)
    q, k, v = torch.randn(9, 4 * 10), torch.randn(9, 20), torch.randn(9, 12)
    ck, cv = (rotary.angles(pos, rotary.frequencies(b, n)) for b, n in ((70.0, 4), (70.0, 6)))
    qr, kr, vr = c.rotate_append(0, q, k, v, ck, cv, 4, 16, slot, pos, 1e-3, True)
    kg, vg = c.gather(0, a, 3, 6, 16)
    assert torch.equal(kg, kr[3:]) and torch.equal(vg, vr[3:]) and float(kg[..., 10:].abs().max()) == 0
    for j in range(9):
        assert torch.allclose(qr[j, :, :10].double(), plain.turn(q[j].view(4, 10).double(), j, 70.0, 4), atol=1e-5)
        assert torch.allclose(kr[j, :, :10].double(), plain.turn(k[j].view(2, 10).double(), j, 70.0, 4), atol=1e-5)
        assert torch.allclose(vr[j, :, :6].double(), plain.turn(plain.rms(v[j].view(2, 6).double(), 1e-3), j, 70.0, 6), atol=1e-5)


@pytest.mark.parametrize("block", [4, 7, 64])
def test_a_standing_out_key_is_seen_up_to_its_blocks_end_only(block):
    n, d = 40, 8
    for at in (0, 3, 4, 6, 7, 13, 14, 27, 28):
        k, q = S.standing_out(n, d, at)
        c = HybridCache([KvShape(1, d, d)], 1, n, page_size=8, dtype=F32, n_pages=5)
        s = c.open()
        c.reserve(s, n)
        pos, slot = torch.arange(n, dtype=torch.int32), torch.full((n,), s, dtype=torch.int32)
        v = torch.randn(n, d)
        c.rotate_append(0, q.float()[None].repeat(n, 1), k.float(), v, None, None, 1, 8, slot, pos, None, False)
        got = c.attention(0, q.float()[None, None].repeat(n, 1, 1), slot, pos, 1.5, n, torch.empty(n, d), block, True)
        for i in range(n):
            see = plain.visible(i, block)
            want = plain.sink_weights(k[see.start:i + 1] @ q * 1.5) @ v[see.start:i + 1].double()
            assert torch.allclose(got[i].double(), want, atol=1e-5)
            seen = at in see
            assert (float((got[i].double() - v[at].double()).abs().max()) < 0.05) == seen


# ------------------------------------------------------------------ configuration and files
def test_configuration_round_trip_and_rejections(tmp_path):
    for name, d in S.cases().items():
        cfg = NufalornConfig.from_dict(d)
        back = json.loads(json.dumps(cfg.to_dict()))
        assert NufalornConfig.from_dict(back) == cfg, name
        for l in back["layers"]:                                    # without the key the checkpoint's shapes decide
            l["mixer"].pop("a_rank", None)
        assert NufalornConfig.from_dict(back, {k: tuple(v.shape) for k, v in random_tensors(cfg).items()}) == cfg, name
    d, cfg, t = S.build("mixed")
    names = cfg.tensor_shapes()
    assert "l3.mix.k" not in names and "l3.mix.q" in names and "l2.norm2" not in names and names["l4.mix.a1"] == (24, 96)

    def change(i, **kw):
        layers = [json.loads(json.dumps(l)) for l in d["layers"]]
        for k, v in kw.items():
            if k in layers[i]:
                layers[i][k] = v
            else:
                layers[i]["mixer"][k] = v
        return {**d, "layers": layers}
    for bad, words in ((change(0, type="other"), "mixer"), (change(0, mlp={"kind": "moe"}), "feed-forward"), (change(0, heads=5), "groups"),
                       (change(3, kv_from=1), "keys and values"), (change(3, kv_from=4), "keys and values"), (change(3, dim=32), "keys and values"),
                       (change(0, rot={"base": 10.0, "dims": 26}), "even")):
        with pytest.raises(ValueError, match=words):
            NufalornConfig.from_dict(bad)
    registry.save_folder(str(tmp_path / "m"), cfg, t)
    m = registry.load_folder(str(tmp_path / "m"), "cpu", F32)
    assert isinstance(m, Nufalorn) and m.cfg == cfg
    with pytest.raises(ValueError, match="missing"):
        Nufalorn(cfg, {k: v for k, v in t.items() if k != "l1.mix.lower"})


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_prompt_portions_and_single_tokens_match_the_restatement(name):
    d, cfg, t = S.build(name)
    n = 85
    toks = S.tokens(n, cfg.vocab_size, 1)
    want = S.expect(d, t, toks)
    e = S.engine(cfg, t, "cpu", F32, page_size=16)
    for cuts in ([(0, n)], S.singles(0, n), S.portions(n, [33, 2, 5]), S.portions(n, [2])):
        S.assert_close(S.feed(e, toks, cuts), want, F32, cuts[:3])
    b = S.engine(cfg, t, "cpu", torch.bfloat16, page_size=64)
    for cuts in ([(0, n)], S.portions(n, [40, 1, 34])):
        S.assert_close(S.feed(b, toks, cuts), want, torch.bfloat16, cuts[:3])


def test_every_layer_of_the_stream_matches():
    d, cfg, t = S.build("mixed", 3)
    toks = S.tokens(41, cfg.vocab_size, 4)
    want, got = [], []
    plain.forward(d, t, toks, keep=want)
    e = S.engine(cfg, t, "cpu", F32)
    e.step([(e.open(), toks, [])], keep=got)
    assert len(got) == len(want) == 5
    for i, (a, b) in enumerate(zip(got, want)):
        assert torch.allclose(a.double(), b, atol=2e-4), i


def test_sequences_in_one_batch_do_not_touch_each_other_and_pages_and_slots_are_used_again():
    d, cfg, t = S.build("mixed", 5)
    seqs = [S.tokens(n, cfg.vocab_size, 10 + n) for n in (60, 3, 47, 18)]
    want = [S.expect(d, t, s) for s in seqs]
    e = S.engine(cfg, t, "cpu", F32, page_size=8, pool=136)
    for _ in range(3):
        slots = [e.open() for _ in seqs]
        at, got = [0] * 4, [[] for _ in seqs]
        for row in [(50, 2, 0, 17), (1, 1, 45, 1), (9, 0, 2, 0)]:
            part = [(i, n) for i, n in enumerate(row) if n]
            out = e.step([(slots[i], seqs[i][at[i]:at[i] + n], list(range(n))) for i, n in part])
            for i, n in part:
                got[i].append(out[:n])
                out = out[n:]
                at[i] += n
        for i in (2, 0, 3, 1):
            assert at[i] == len(seqs[i])
            S.assert_close(torch.cat(got[i]).double(), want[i], F32, i)
            e.close(slots[i])


def test_scheduler_generates_greedily_with_more_requests_than_slots():
    d, cfg, t = S.build("mixed", 7)
    prompts = [S.tokens(n, cfg.vocab_size, n) for n in (5, 40, 1, 54, 12, 9)]
    want = [S.greedy(d, t, p, 5) for p in prompts]
    e = S.engine(cfg, t, "cpu", F32, slots=3, page_size=8, pool=120)
    s = Scheduler(e, step_tokens=16)
    reqs = [s.add(p, 5) for p in prompts]
    s.run()
    assert [r.tokens for r in reqs] == want
    assert e.free_slots() == 3 and e.cache.free_pages() == e.cache.n_pages - 1
    assert generate(e, prompts[:2], 5) == want[:2]


def test_speculative_decoder_takes_back_states():
    d, cfg, t = S.build("mixed", 7)
    other = random_tensors(cfg, 8)
    mix = {k: (0.9 * v.float() + 0.1 * other[k].float()).to(v.dtype) for k, v in t.items()}        # a draft that is sometimes wrong
    prompts = torch.tensor([S.tokens(39, cfg.vocab_size, 1), S.tokens(39, cfg.vocab_size, 2)])
    want = [S.greedy(d, t, p.tolist(), 8) for p in prompts]
    m = Nufalorn(cfg, t, "cpu", F32)
    dec = SpeculativeDecoder(StackEngine(Nufalorn(cfg, mix, "cpu", F32), 2, 128), StackEngine(m, 2, 128), gamma=3, temperature=0.0)
    seqs, stats = dec.generate(prompts, 8)
    assert [s[39:47] for s in seqs] == want and 0 < stats.acceptance_rate < 1
    dec = SpeculativeDecoder(StackEngine(m, 2, 128), StackEngine(m, 2, 128), gamma=3, temperature=0.0)
    seqs, stats = dec.generate(prompts, 8)
    assert [s[39:47] for s in seqs] == want and stats.acceptance_rate == 1.0
    with pytest.raises(ValueError, match="take back"):
        SpeculativeDecoder(StackEngine(m, 2, 128), StackEngine(m, 2, 128), gamma=16)


def test_trace_replay_and_command_line(tmp_path):
    from cogito_b200.cli import main
    d, cfg, t = S.build("mixed", 7)
    folder = str(tmp_path / "model")
    registry.save_folder(folder, cfg, t)
    toks, other = S.tokens(50, cfg.vocab_size, 1), S.tokens(6, cfg.vocab_size, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:42], "want": [3, 41]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": other, "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[42:], "want": [7]}], "end": ["a"]}]
    e = S.engine(cfg, t, "cpu", F32)
    done = []
    trace.replay(e, io.StringIO("\n".join(json.dumps(s) for s in steps)), str(tmp_path), done.append)
    want = S.expect(d, t, toks)
    assert done == [0, 1, 2] and not (tmp_path / "1.f32").exists() and e.free_slots() == 4
    got = [np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, cfg.vocab_size) for i in (0, 2)]
    S.assert_close(torch.from_numpy(np.concatenate(got)).double(), want[[3, 41, 49]], F32)
    prompts = [S.tokens(n, cfg.vocab_size, n) for n in (4, 41, 7)]
    (tmp_path / "p.json").write_text(json.dumps(prompts))
    out = main(["generate", "device=cpu", f"model.path={folder}", "generate.dtype=float32", "generate.new_tokens=4", f"generate.out={tmp_path}/o.json",
                f"generate.prompts={tmp_path}/p.json", "generate.slots=2"])
    assert out["generated"] == 12
    assert json.loads((tmp_path / "o.json").read_text()) == [p + S.greedy(d, t, p, 4) for p in prompts]
