"""Surelorn on the host path: configuration, files, cache and slots, portions and batches, scheduler, command line,
trace replay - against the slow restatement in plain_surelorn.py."""
import io
import json

import numpy as np
import pytest
import torch

import plain_surelorn as plain
import surelorn_cases as S
from cogito_b200.io.safetensors import load_safetensors, save_safetensors
from cogito_b200.models import registry
from cogito_b200.models.surelorn import Surelorn, SurelornConfig, random_tensors, save_folder
from cogito_b200.ops import moe as X
from cogito_b200.ops import stream as R
from cogito_b200.serve import trace
from cogito_b200.serve.engine import SpeculativeDecoder
from cogito_b200.serve.kv_cache import PagedLatentCache
from cogito_b200.serve.scheduler import Scheduler, generate
from cogito_b200.serve.stack import StackEngine

F32 = torch.float32


# ------------------------------------------------------------------ the restatement itself
def test_plain_attention_sees_exactly_the_earlier_positions_and_expands_per_head():
    torch.manual_seed(0)
    m = S.mixer(2, 4, 3, 5, 6, 0.7)
    w = {"dq": torch.randn(5, 8), "dq.norm": torch.rand(5), "uq": torch.randn(8, 5), "dkv": torch.randn(6, 8), "dkv.norm": torch.rand(6),
         "uk": torch.randn(8, 6), "uv": torch.randn(6, 6), "o": torch.randn(8, 6)}
    w = {k: v.double() for k, v in w.items()}
    x = torch.randn(9, 8).double()
    y = plain.latent_attention(x, w, m, 1e-6)
    for i in (0, 4, 8):                                   # later tokens change nothing, earlier ones do
        assert torch.allclose(plain.latent_attention(x[:i + 1], w, m, 1e-6)[i], y[i])
    x2 = x.clone()
    x2[2] += 1
    y2 = plain.latent_attention(x2, w, m, 1e-6)
    assert torch.equal(y2[:2], y[:2]) and not torch.allclose(y2[8], y[8])


def test_plain_router_keeps_groups_by_their_best_choice_score_and_weighs_without_the_correction():
    logits = torch.log(torch.tensor([0.30, 0.01, 0.20, 0.19, 0.02, 0.28], dtype=torch.float64))
    # the correction makes output 4 the best; groups {0,1} {2,3} {4,5}; two kept
    corr = torch.tensor([-0.5, -0.9, 0.0, 0.0, 0.5, -0.9], dtype=torch.float64)
    got = plain.choose(logits, corr, {"groups": {"count": 3, "keep": 2}, "top": 3})
    assert [i for i, _ in got] == [4, 2, 3]
    assert [round(float(v), 6) for _, v in got] == [round(v / 0.41, 6) for v in (0.02, 0.20, 0.19)]
    # output 5 chooses at -0.62: below zero, and still ahead of everything in the group that was dropped
    corr2 = torch.tensor([-0.5, -0.9, 0.0, -3.0, 0.5, -0.9], dtype=torch.float64)
    assert [i for i, _ in plain.choose(logits, corr2, {"groups": {"count": 3, "keep": 2}, "top": 4})] == [4, 2, 5, 3]


# ------------------------------------------------------------------ mechanisms, host form
@pytest.mark.parametrize("experts,identity,top,groups,keep", [(6, 2, 3, 4, 2), (5, 0, 2, 1, 1), (30, 10, 8, 8, 3), (4, 4, 1, 2, 1)])
def test_routing_matches_the_restatement(experts, identity, top, groups, keep):
    torch.manual_seed(experts)
    O = experts + identity
    logits, corr = torch.randn(40, O) * 2, torch.randn(O) * 0.3 - 0.2
    r = X.route(logits, corr, experts, top, groups, keep)
    for t in range(40):
        want = plain.choose(logits[t].double(), corr.double(), {"groups": {"count": groups, "keep": keep}, "top": top})
        assert r.idx[t].tolist() == [i for i, _ in want]
        assert torch.allclose(r.weight[t].double(), torch.stack([v for _, v in want]), atol=1e-6)
        assert [v >= 0 for v in r.row_of[t].tolist()] == [i < experts for i, _ in want]


def test_embedding_and_stream_update():
    torch.manual_seed(0)
    for width in (10, 7):                                 # an odd width ends with a sine
        table = torch.randn(20, width)
        pos = torch.tensor([0, 1, 5, 4000], dtype=torch.int32)
        x, h = R.embed_sinusoid(torch.tensor([3, 19, 0, 7]), pos, table, 2.5, R.sinusoid_frequencies(width))
        want = table[[3, 19, 0, 7]].double() * 2.5 + plain.sinusoid(pos.tolist(), width)
        assert torch.allclose(x.double(), want, atol=1e-6) and torch.equal(h, x)
    y, w = torch.randn(4, 7), torch.rand(7)
    pairs = torch.randn(3, 7)
    row_of, weight = torch.tensor([[0, -1], [2, 1], [-1, -1], [1, 0]], dtype=torch.int32), torch.rand(4, 2)
    v = y.clone()
    for t in range(4):
        for k in range(2):
            r = int(row_of[t, k])
            v[t] += weight[t, k] * (pairs[r] if r >= 0 else x[t])
    want = x + plain.rms(v.double(), w.double(), 1e-3).float()
    R.stream_update(x, y, w, 1e-3, F32, pairs, row_of, weight)
    assert torch.allclose(x, want, atol=1e-5)


def test_latent_cache_places_frees_and_refuses():
    c = PagedLatentCache([4, 6], 3, 20, page_size=4, dtype=F32, n_pages=6)
    a, b = c.open(), c.open()
    c.reserve(a, 5)
    c.reserve(b, 12)
    assert c.free_pages() == 1 and set(c._owned[a]).isdisjoint(c._owned[b])
    with pytest.raises(RuntimeError, match="exhausted"):
        c.reserve(a, 13)
    with pytest.raises(ValueError, match="exceeds"):
        c.reserve(a, 21)
    slot, pos = torch.full((5,), a, dtype=torch.int32), torch.arange(5, dtype=torch.int32)
    lat = torch.randn(5, 3 + 6)
    cq, cc = c.norm_append(1, lat, torch.ones(3), torch.full((6,), 2.0), 1e-6, slot, pos, True)
    assert torch.allclose(c.gather(1, a, 5), plain.rms(lat[:, 3:].double(), torch.full((6,), 2.0).double(), 1e-6).float(), atol=1e-6)
    assert torch.allclose(cq, plain.rms(lat[:, :3].double(), torch.ones(3).double(), 1e-6).float(), atol=1e-6) and torch.equal(c.gather(1, a, 5), cc)
    pages = list(c._owned[b])
    c.close(b)
    d = c.open()
    c.reserve(d, 12)                                      # the pages serve another sequence
    assert d == b and set(c._owned[d]) == set(pages)
    c.open()
    with pytest.raises(RuntimeError, match="no free"):
        c.open()


# ------------------------------------------------------------------ configuration and files
def test_configuration_round_trip_and_rejections(tmp_path):
    for name, d in S.cases().items():
        cfg = SurelornConfig.from_dict(d)
        assert SurelornConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg, name
    d = S.cases()["mixed"]
    cfg = SurelornConfig.from_dict(d)
    assert [cfg.home(i) for i in range(6)] == [0, 1, 0, 3, 3, 0] and cfg.layers[3].mlp is None
    assert "l2.norm1" not in cfg.tensor_shapes() and "l3.norm2" not in cfg.tensor_shapes()
    with pytest.raises(ValueError, match="mixer"):
        SurelornConfig.from_dict({**d, "layers": [{**d["layers"][0], "type": "other"}]})
    with pytest.raises(ValueError, match="groups"):
        SurelornConfig.from_dict({**d, "layers": [S.layer(d["layers"][0]["mixer"], S.moe(8, 6, 3, 2, (4, 1)))]})
    with pytest.raises(ValueError, match="weights_of"):
        SurelornConfig.from_dict({**d, "layers": [S.layer(d["layers"][0]["mixer"], None, 0)]})
    with pytest.raises(ValueError, match="sizes differ"):
        SurelornConfig.from_dict({**d, "layers": [d["layers"][0], S.layer(d["layers"][0]["mixer"], None, 0)]})
    t = random_tensors(cfg)
    save_folder(str(tmp_path / "m"), cfg, t)
    back = load_safetensors(str(tmp_path / "m" / "model.safetensors"))
    assert back.keys() == t.keys() and all(torch.equal(back[k], t[k]) for k in t)
    m = registry.load_folder(str(tmp_path / "m"), "cpu", F32)
    assert isinstance(m, Surelorn) and m.cfg == cfg
    with pytest.raises(ValueError, match="missing"):
        Surelorn(cfg, {k: v for k, v in t.items() if k != "head"})
    (tmp_path / "m" / "config.json").write_text('{"architecture": "Nothing"}')
    with pytest.raises(ValueError, match="Nothing"):
        registry.load_folder(str(tmp_path / "m"), "cpu")


def test_safetensors_types_and_damaged_files(tmp_path):
    t = {"a": torch.arange(5, dtype=torch.int32), "b": torch.randn(2, 3), "c": torch.randn(4).bfloat16(), "d": torch.tensor([True, False]),
         "e": torch.zeros(0, 4), "f": torch.tensor(2.5)}
    p = str(tmp_path / "x.safetensors")
    save_safetensors(p, t)
    back = load_safetensors(p)
    assert all(torch.equal(back[k], t[k]) and back[k].dtype == t[k].dtype for k in t)
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-3])
    with pytest.raises(ValueError, match="place"):
        load_safetensors(p)
    open(p, "wb").write(b"\xff" * 20)
    with pytest.raises(ValueError):
        load_safetensors(p)


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_prompt_portions_and_single_tokens_match_the_restatement(name):
    d, cfg, t = S.build(name)
    toks = S.tokens(75, cfg.vocab_size, 1)
    want = S.expect(d, t, toks)
    e = S.engine(cfg, t, "cpu", F32, page_size=16)
    for cuts in ([(0, 75)], [(i, 1) for i in range(75)], S.portions(75, [33, 2, 5]), S.portions(75, [2])):
        S.assert_close(S.feed(e, toks, cuts), want, F32, cuts[:3])
    b = S.engine(cfg, t, "cpu", torch.bfloat16, page_size=64)      # the prompt form with padded heads
    for cuts in ([(0, 75)], S.portions(75, [40, 1, 34])):
        S.assert_close(S.feed(b, toks, cuts), want, torch.bfloat16, cuts[:3])


def test_every_layer_of_the_stream_matches():
    d, cfg, t = S.build("mixed", 3)
    toks = S.tokens(21, cfg.vocab_size, 4)
    want, got = [], []
    plain.forward(d, t, toks, keep=want)
    e = S.engine(cfg, t, "cpu", F32)
    e.step([(e.open(), toks, [])], keep=got)
    assert len(got) == len(want) == 6
    for i, (a, b) in enumerate(zip(got, want)):
        assert torch.allclose(a.double(), b, atol=2e-4), i


def test_sequences_in_one_batch_do_not_touch_each_other_and_pages_are_used_again():
    d, cfg, t = S.build("mixed", 5)
    seqs = [S.tokens(n, cfg.vocab_size, 10 + n) for n in (50, 3, 37, 18)]
    want = [S.expect(d, t, s) for s in seqs]
    e = S.engine(cfg, t, "cpu", F32, page_size=8, pool=128)
    for _ in range(3):                                    # later rounds run on pages that others have filled
        slots = [e.open() for _ in seqs]
        at, got = [0] * 4, [[] for _ in seqs]
        plan = [(40, 2, 0, 17), (1, 1, 35, 1), (9, 0, 2, 0)]
        for row in plan:
            part = [(i, n) for i, n in enumerate(row) if n]
            out = e.step([(slots[i], seqs[i][at[i]:at[i] + n], list(range(n))) for i, n in part])
            for i, n in part:
                got[i].append(out[:n])
                out = out[n:]
                at[i] += n
        for i in range(4):
            assert at[i] == len(seqs[i])
            S.assert_close(torch.cat(got[i]).double(), want[i], F32, i)
            e.close(slots[i])
    with pytest.raises(ValueError, match="one entry"):
        s = e.open()
        e.step([(s, [1], []), (s, [2], [])])
    with pytest.raises(ValueError, match="token ids"):
        e.step([(s, [cfg.vocab_size], [])])


def _greedy(d, t, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(S.expect(d, t, seq)[-1].argmax()))
    return seq[len(prompt):]


def test_scheduler_generates_greedily_with_more_requests_than_slots():
    d, cfg, t = S.build("mixed", 7)
    prompts = [S.tokens(n, cfg.vocab_size, n) for n in (5, 30, 1, 44, 12, 9, 3)]
    want = [_greedy(d, t, p, 6) for p in prompts]
    e = S.engine(cfg, t, "cpu", F32, slots=3, page_size=8, pool=96)
    s = Scheduler(e, step_tokens=16)                      # prompts are cut, decoding runs beside them
    reqs = [s.add(p, 6) for p in prompts]
    s.run()
    assert [r.tokens for r in reqs] == want
    assert e.free_slots() == 3 and e.cache.free_pages() == e.cache.n_pages - 1
    assert generate(e, prompts[:2], 6) == want[:2]
    stop = s.add(prompts[0], 6, stop_token=want[0][2])
    s.run()
    assert stop.tokens == want[0][:want[0].index(want[0][2]) + 1]
    with pytest.raises(ValueError, match="exceeds"):
        s.add([1] * 2000, 4)


def test_speculative_decoder_runs_on_the_stack_engine():
    d, cfg, t = S.build("mixed", 7)
    prompts = torch.tensor([S.tokens(9, cfg.vocab_size, 1), S.tokens(9, cfg.vocab_size, 2)])
    want = [_greedy(d, t, p.tolist(), 8) for p in prompts]
    m = Surelorn(cfg, t, "cpu", F32)
    dec = SpeculativeDecoder(StackEngine(m, 2, 128), StackEngine(m, 2, 128), gamma=3, temperature=0.0)
    seqs, stats = dec.generate(prompts, 8)
    assert [s[9:17] for s in seqs] == want and stats.acceptance_rate == 1.0


def test_trace_replay_and_command_line(tmp_path):
    from cogito_b200.cli import main
    d, cfg, t = S.build("mixed", 7)
    folder = str(tmp_path / "model")
    save_folder(folder, cfg, t)
    toks, other = S.tokens(20, cfg.vocab_size, 1), S.tokens(6, cfg.vocab_size, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:12], "want": [3, 11]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": other, "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[12:], "want": [7]}], "end": ["a"]}]
    e = S.engine(cfg, t, "cpu", F32)
    done = []
    trace.replay(e, io.StringIO("\n".join(json.dumps(s) for s in steps)), str(tmp_path), done.append)
    want = S.expect(d, t, toks)
    assert done == [0, 1, 2] and not (tmp_path / "1.f32").exists() and e.free_slots() == 4
    got = np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(2, -1)
    S.assert_close(torch.from_numpy(got).double(), want[[3, 11]], F32)
    S.assert_close(torch.from_numpy(np.fromfile(tmp_path / "2.f32", dtype="<f4")[None]).double(), want[[19]], F32)

    prompts = [S.tokens(n, cfg.vocab_size, n) for n in (4, 11, 7)]
    (tmp_path / "p.json").write_text(json.dumps(prompts))
    base = ["generate", "device=cpu", f"model.path={folder}", "generate.dtype=float32", "generate.new_tokens=5", f"generate.out={tmp_path}/o.json"]
    out = main(base + [f"generate.prompts={tmp_path}/p.json", "generate.slots=2"])
    assert out["generated"] == 15
    assert json.loads((tmp_path / "o.json").read_text()) == [p + _greedy(d, t, p, 5) for p in prompts]
    out = main(base + [f"generate.draft_path={folder}", "generate.batch=2", "generate.prompt_len=6"])
    seqs = json.loads((tmp_path / "o.json").read_text())
    assert all(s[6:11] == _greedy(d, t, s[:6], 5) for s in seqs)


def test_the_serving_subset_of_the_kernels_has_what_the_engine_calls(tmp_path):
    """A checkout that only serves compiles part of the library: it must load, and every function that the modules
    on the serving path name must be in it."""
    import ctypes
    import re
    import subprocess
    import sys
    from pathlib import Path

    from cogito_b200 import build
    root = Path(__file__).resolve().parent.parent
    if not all((build.BUILD_DIR / "kernels" / f"{n}.o").exists() for n in build.SERVE_SOURCES):
        pytest.skip("kernel objects have not been compiled here")
    so = build.build_serving_kernels(out=tmp_path / "serve.so")
    lib = ctypes.CDLL(str(so))
    named = set()
    for f in ("ops/stream.py", "ops/moe.py", "ops/linear.py", "ops/gemm.py", "ops/recurrence.py", "ops/rotary.py", "serve/kv_cache.py",
              "serve/hybrid_cache.py", "serve/sampling.py"):
        named |= set(re.findall(r"\.(cgk_\w+)\(", (root / "cogito_b200" / f).read_text()))
    assert len(named) > 15 and not [n for n in named if not hasattr(lib, n)]
    # the bindings accept a library without the training kernels
    code = ("import sys; sys.path.insert(0, sys.argv[1]); from pathlib import Path; from cogito_b200.ops import _lib, attention; "
            "_lib._LIB_PATH = Path(sys.argv[2]); L = attention._fns(); print(L.cgk_version(), bool(L.cgk_flash_forward.argtypes))")
    r = subprocess.run([sys.executable, "-c", code, str(root), str(so)], capture_output=True, text=True)
    assert r.returncode == 0 and r.stdout.split()[1] == "True", r.stderr
