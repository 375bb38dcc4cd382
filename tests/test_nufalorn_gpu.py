"""Nufalorn on a B200: each kernel against a slow restatement, and the engine (bf16 and fp32) against plain_nufalorn.py:
prompts, portions, decoding, batches, reused pages and slots, block edges, sinks, sampling and graphs."""
import math
from types import SimpleNamespace

import pytest
import torch

import nufalorn_cases as S
import plain_nufalorn as plain
from cogito_b200.models import registry
from cogito_b200.ops import _lib
from cogito_b200.ops import misc as M
from cogito_b200.ops import recurrence as R
from cogito_b200.ops import rotary
from cogito_b200.ops import stream as X
from cogito_b200.ops.attention import flash_forward
from cogito_b200.ops.linear import gated_linear
from cogito_b200.serve.hybrid_cache import HybridCache, KvShape

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


def ints(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------ row kernels
@pytest.mark.parametrize("base,dims", [(10000.0, 64), (1e6, 10), (3.0, 2)])
def test_angles(base, dims):
    pos = torch.tensor([0, 1, 2, 63, 1000, 4097, 131071], dtype=torch.int32)
    cs = rotary.angles(pos.to(DEV), rotary.frequencies(base, dims, DEV)).cpu().double()
    for i, p in enumerate(pos.tolist()):
        for j in range(dims // 2):
            a = p * base ** (-2.0 * j / dims)
            assert abs(float(cs[i, j, 0]) - math.cos(a)) < 1e-6 and abs(float(cs[i, j, 1]) - math.sin(a)) < 1e-6


@pytest.mark.parametrize("D", [96, 352, 4096, 8192, 130, 33])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_stream_norms(D, dtype):
    N = 11
    table, ids = rand(20, D, seed=1, dtype=dtype), torch.randint(0, 20, (N,))
    w1, w2 = torch.rand(D) + 0.5, torch.rand(D) + 0.5
    x = torch.empty(N, D, device=DEV)
    h1, h2 = X.stream_norms(x, 1e-4, dtype, w1.to(DEV), w2.to(DEV), ids=ids.to(DEV), table=table.to(DEV))
    assert torch.equal(x.cpu(), table[ids].float())
    tol = 1e-5 if dtype == F32 else 4e-2
    for y_dt in {dtype, F32}:
        before, y = x.cpu().double(), rand(N, D, seed=2, dtype=y_dt, scale=3.0)
        h1, h2 = X.stream_norms(x, 1e-4, dtype, w1.to(DEV), w2.to(DEV), y=y.to(DEV), mult=0.6)
        want = before + 0.6 * y.double()
        assert torch.allclose(x.cpu().double(), want, atol=1e-5)
        n = plain.rms(want, 1e-4)
        assert h1.dtype == dtype and torch.allclose(h1.cpu().double(), n * w1, atol=tol) and torch.allclose(h2.cpu().double(), n * w2, atol=tol)
    none, h2 = X.stream_norms(x, 1e-4, dtype, None, w2.to(DEV))
    assert none is None and torch.allclose(h2.cpu().double(), n * w2, atol=tol)
    before, y = x.cpu(), rand(N, D, seed=3)
    assert X.stream_norms(x, 1e-4, F32, y=y.to(DEV), mult=2.0) == (None, None) and torch.allclose(x.cpu(), before + 2 * y, atol=1e-5)


def test_softcap_and_relu_gate():
    x = rand(7, 333, scale=40.0)
    got = X.softcap(x.to(DEV), 9.0).cpu().double()
    assert float((got - 9.0 * torch.tanh(x.double() / 9.0)).abs().max()) < 2e-6 * 9
    for dtype, rows, F in [(BF, 5, 64), (BF, 300, 24), (BF, 9, 13), (F32, 6, 10)]:
        gu = rand(rows, 2 * F, dtype=dtype)
        want = torch.clamp(gu[:, :F].double(), min=0) * gu[:, F:].double()
        for wide in (F, F + 40):
            out = torch.zeros(rows, wide, dtype=dtype, device=DEV)
            M.gated(gu.to(DEV), "relu", out[:, :F])
            assert torch.allclose(out[:, :F].cpu().double(), want, atol=1e-6, rtol=1e-2 if dtype == BF else 1e-6) and float(out[:, F:].abs().sum()) == 0
    for rows in (1, 3, 8, 9):
        a, w = rand(rows, 72, dtype=BF), rand(2 * 50, 72, seed=3, dtype=BF, scale=0.2)
        want = torch.clamp(a.double() @ w[:50].double().T, min=0) * (a.double() @ w[50:].double().T)
        out = torch.zeros(rows, 56, dtype=BF, device=DEV)
        gated_linear(a.to(DEV), w.to(DEV), "relu", out[:, :50])
        assert float((out[:, :50].cpu().double() - want).abs().max()) < 2e-2 * float(want.abs().max())


# ------------------------------------------------------------------ keys and values
@pytest.mark.parametrize("H,G,dim,vdim,rot,page", [(6, 2, 24, 40, 16, 16), (4, 2, 64, 64, 64, 64), (5, 5, 18, 10, 6, 7), (16, 4, 128, 128, 128, 64), (2, 1, 144, 160, 20, 64)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_rotate_append_and_gather(H, G, dim, vdim, rot, page, dtype):
    N, first = 50, 13
    c = HybridCache([KvShape(G, dim, vdim)], 2, 128, page, DEV, dtype, n_pages=20)
    c._free_pages = torch.randperm(20, generator=torch.Generator().manual_seed(1)).tolist()
    s = c.open()
    c.reserve(s, first + N)
    pos = torch.arange(first, first + N, dtype=torch.int32)
    x = rand(N, H * dim + G * (dim + vdim) + 8, seed=2, dtype=dtype)
    q, k, v = x[:, :H * dim], x[:, H * dim:(H + G) * dim], x[:, (H + G) * dim:(H + G) * dim + G * vdim]
    wide = max((max(dim, vdim) + 7) // 8 * 8, 64)
    ck, cv = (rotary.angles(pos.to(DEV), rotary.frequencies(500.0, n, DEV)) for n in (rot, vdim))
    xd = x.to(DEV)
    qd, kd, vd = xd[:, :H * dim], xd[:, H * dim:(H + G) * dim], xd[:, (H + G) * dim:(H + G) * dim + G * vdim]
    qr, kr, vr = c.rotate_append(0, qd, kd, vd, ck, cv, H, wide, ints([s] * N), pos.to(DEV), 1e-4, True)
    kg, vg = c.gather(0, s, first, N, wide)
    assert torch.equal(kg, kr) and torch.equal(vg, vr)
    tol = 1e-5 if dtype == F32 else 2e-2
    for i in range(0, N, 7):
        p = first + i
        for got, want in ((qr, plain.turn(q[i].double().view(H, dim), p, 500.0, rot)), (kr, plain.turn(k[i].double().view(G, dim), p, 500.0, rot)),
                          (vr, plain.turn(plain.rms(v[i].double().view(G, vdim), 1e-4), p, 500.0, vdim))):
            n = want.shape[1]
            assert torch.allclose(got[i, :, :n].cpu().double(), want, atol=tol, rtol=tol) and float(got[i, :, n:].abs().sum()) == 0
    only, none, _ = c.rotate_append(0, qd, None, None, ck, None, H, wide, ints([s] * N), pos.to(DEV), None, True)
    assert none is None and torch.equal(only, qr)


def _kv(G, dim, vdim, lengths, dtype, page=64, seed=0, spare=3):
    """A cache whose sequences own shuffled pages, filled with random keys and values (spare pages hold huge ones)."""
    g = torch.Generator().manual_seed(seed)
    pages = sum(-(-n // page) for n in lengths) + spare
    c = HybridCache([KvShape(G, dim, vdim)], len(lengths), max(lengths), page, DEV, dtype, n_pages=pages)
    _, kp, vp = c.kv[0]
    kp[..., :dim] = 77.0
    vp[..., :vdim] = 77.0
    c._free_pages = torch.randperm(pages, generator=g).tolist()
    data = []
    for n in lengths:
        s = c.open()
        c.reserve(s, n)
        k, v = torch.randn(n, G, dim, generator=g).to(dtype), torch.randn(n, G, vdim, generator=g).to(dtype)
        at = torch.arange(n, device=DEV)
        pg = c.page_table[s, at // page].long()
        kp[pg, :, at % page, :dim], vp[pg, :, at % page, :vdim] = k.to(DEV), v.to(DEV)
        data.append((s, k.double(), v.double()))
    return c, data


def _attend(q, k, v, p, scale, block, sink, turn_base=None):
    """q [H, dim] of one token at position p."""
    H, G = q.shape[0], k.shape[1]
    see = plain.visible(p, block or 10**9)
    out = []
    for h in range(H):
        s = k[see.start:p + 1, h * G // H] @ q[h].double() * scale
        out.append((plain.sink_weights(s) if sink else torch.softmax(s, -1)) @ v[see.start:p + 1, h * G // H])
    out = torch.stack(out)
    return out if turn_base is None else plain.turn(out, p, turn_base, out.shape[1], -1)


def _padded(q, wide):
    return torch.nn.functional.pad(q, (0, wide - q.shape[-1])).to(DEV)


@pytest.mark.parametrize("H,G,dim,vdim", [(12, 1, 64, 64), (6, 2, 24, 40), (5, 5, 18, 10), (16, 4, 128, 128), (7, 1, 32, 128), (4, 2, 144, 160), (2, 1, 520, 8), (3, 1, 8, 1000)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_attention_of_single_tokens_over_pages(H, G, dim, vdim, dtype):
    lengths = [1, 2, 63, 64, 65, 128, 129, 700]
    for page in (64, 24):
        c, data = _kv(G, dim, vdim, lengths, dtype, page, seed=dim)
        places = [(i, n - 1) for i, n in enumerate(lengths)] + [(7, 0), (7, 255), (7, 256), (7, 511)]
        q = rand(len(places), H, dim, seed=9, dtype=dtype)
        wide, scale = (dim + 7) // 8 * 8, 1.5 * dim ** -0.5
        slot, pos = ints([data[k][0] for k, _ in places]), ints([p for _, p in places])
        turn = rotary.angles(pos, rotary.frequencies(90.0, vdim, DEV))
        for block, sink, turned in ((0, False, False), (0, True, True), (100, True, True), (64, False, True), (1, True, False)):
            want = torch.stack([_attend(q[i], *data[k][1:], p, scale, block, sink, 90.0 if turned else None).reshape(-1) for i, (k, p) in enumerate(places)])
            for splits in (0, 1, 5):
                out = torch.zeros(len(places), H * vdim + 8, dtype=dtype, device=DEV)
                c.attention(0, _padded(q, wide), slot, pos, scale, 700, out[:, :H * vdim], block, sink, turn if turned else None, splits)
                err = float((out[:, :H * vdim].cpu().double() - want).abs().max())
                assert err < (1e-5 if dtype == F32 else 1e-2) * float(want.abs().max()), (block, sink, splits, err)


@pytest.mark.parametrize("H,G,dim,vdim,wide", [(10, 2, 64, 64, 64), (6, 2, 24, 40, 64), (16, 4, 128, 128, 128), (3, 3, 72, 20, 128), (2, 1, 50, 34, 64)])
def test_prompt_attention_with_blocks_sink_and_turned_results(H, G, dim, vdim, wide):
    for B, T, begin, block, sink in ((1, 300, 0, 37, True), (2, 260, 0, 190, True), (1, 129, 128, 64, True), (1, 40, 600, 600, False), (1, 520, 0, 0, True),
                                     (1, 257, 256, 256, True), (1, 33, 0, 1, True), (3, 64, 0, 129, True), (1, 700, 40, 40, False)):
        q, k, v = (rand(B, n, h, d, seed=s, dtype=BF) for n, h, d, s in ((T, H, dim, 1), (T + begin, G, dim, 2), (T + begin, G, vdim, 3)))
        pos = torch.arange(begin, begin + T, dtype=torch.int32)
        turn = rotary.angles(pos.to(DEV), rotary.frequencies(40.0, vdim, DEV))[None].expand(B, -1, -1, -1).contiguous()
        rows = torch.zeros(B, T, H * vdim + 8, dtype=BF, device=DEV)
        scale = 2.0 * dim ** -0.5
        flash_forward(_padded(q, wide), _padded(k, wide), _padded(v, wide), causal=True, scale=scale, out=rows[..., :H * vdim].unflatten(-1, (H, vdim)), block=block,
                      sink=sink, turn=turn)
        for b in range(B):
            for i in sorted({0, 1, 36, 37, 38, T // 2, T - 2, T - 1} & set(range(T))):
                want = _attend(q[b, i], k[b].double(), v[b].double(), begin + i, scale, block, sink, 40.0)
                err = float((rows[b, i, :H * vdim].cpu().double() - want.reshape(-1)).abs().max())
                assert err < 2e-2 * max(1.0, float(want.abs().max())), (B, T, begin, block, b, i, err)


@pytest.mark.parametrize("block", [64, 100, 128, 0])
def test_one_standing_out_key_is_seen_up_to_its_blocks_end_only(block):
    n, d = 420, 64
    for at in (0, 1, 63, 64, 99, 100, 127, 128, 199, 200, 255, 256, 299, 300, n - 1):
        k, q = S.standing_out(n, d, at)
        k, qq = k.to(BF)[:, None], q.to(BF)[None]
        v = rand(n, 1, d, seed=at, dtype=BF)
        near = sorted({max(at - 1, 0), at, min(at + 1, n - 1), n - 1} | ({p for p in ((at // block + 1) * block - 1, (at // block + 1) * block) if p < n} if block else set()))
        want = torch.stack([_attend(qq, k.double(), v.double(), p, 2.0, block, True) for p in near])[:, 0]
        out = torch.empty(1, n, 1, d, dtype=BF, device=DEV)
        flash_forward(qq[None, None].expand(1, n, 1, d).contiguous().to(DEV), k[None].to(DEV), v[None].to(DEV), causal=True, scale=2.0, block=block, sink=True, out=out)
        got = out[0, near, 0].cpu().double()
        assert float((got - want).abs().max()) < 2e-2 * float(want.abs().max()), at
        for dtype in (BF, F32):
            c, [(s, _, _)] = _kv(1, d, d, [n], dtype)
            i = torch.arange(n, device=DEV)
            pg = c.page_table[s, i // 64].long()
            c.kv[0][1][pg, 0, i % 64], c.kv[0][2][pg, 0, i % 64] = k[:, 0].to(DEV, dtype), v[:, 0].to(DEV, dtype)
            o = torch.empty(len(near), d, dtype=dtype, device=DEV)
            c.attention(0, qq.to(DEV, dtype)[None].expand(len(near), 1, d).contiguous(), ints([s] * len(near)), ints(near), 2.0, n, o, block, True)
            assert float((o.cpu().double() - want).abs().max()) < (1e-4 if dtype == F32 else 1e-2) * float(want.abs().max()), (at, dtype)


def test_sink_with_very_small_and_very_large_scores():
    """Scores far below the sink's leave nothing of the values, scores far above it leave nothing to the sink."""
    d = 64
    for sign, block in ((-1.0, 0), (1.0, 50)):
        q, k, v = (rand(1, 140, 1, d, seed=s, dtype=BF).abs() * m for s, m in ((1, 6.0), (2, 6.0 * sign), (3, 1.0)))
        out = torch.empty(1, 140, 1, d, dtype=BF, device=DEV)
        flash_forward(q.to(DEV), k.to(DEV), v.to(DEV), causal=True, scale=0.5, block=block, sink=True, out=out)
        for i in (0, 49, 50, 139):
            want = _attend(q[0, i], k[0].double(), v[0].double(), i, 0.5, block, True)
            assert float((out[0, i].cpu().double() - want).abs().max()) < 2e-2


# ------------------------------------------------------------------ recurrences
def operands(N, H, D, V, mode, seed, dtype, gate, z_shift=0.0, z_scale=2.0):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    rows = torch.zeros(N, 2 * H * D + 2 * H * V + 8, dtype=dtype)
    rows[:] = r(*rows.shape).to(dtype)
    at = [0, H * D, 2 * H * D, 2 * H * D + H * V, 2 * H * D + 2 * H * V]
    q, k, v, gt = (rows[:, at[i]:at[i + 1]] for i in range(4))
    z = torch.zeros(N, H * D + 8)
    z[:] = z_scale * r(N, H * D + 8) + z_shift
    low = 0.9 * torch.rand(H * D, generator=g) if mode == R.BOUNDED else None
    if low is not None:
        low[::3] = 0.0
    return R.Operands(q, k if mode == R.ROOT else None, v, gt if gate else None, z[:, :H * D], r(H * D), low, 1 + 0.2 * r(V)), (rows, z)


def to_dev(x, back):
    rows, z = (t.to(DEV) for t in back)
    def same(t):
        if t is None:
            return None
        src, base = (rows, back[0]) if t.dtype == back[0].dtype and t.data_ptr() >= back[0].data_ptr() and t.data_ptr() < back[0].data_ptr() + back[0].nbytes else (z, back[1])
        off = (t.data_ptr() - base.data_ptr()) // t.element_size()
        return src[:, off:off + t.shape[1]]
    dev = lambda t: None if t is None else t.to(DEV)
    return R.Operands(same(x.q), same(x.k), same(x.v), same(x.gate), same(x.z), dev(x.bias), dev(x.low), dev(x.w))


def plain_advance(rule, x, rows):
    T, H, D, V = len(rows), rule.heads, rule.dim, rule.vdim
    z = (x.z[rows] + x.bias).double()
    if rule.mode == R.ROOT:
        a, k = plain.sigmoid(z) ** (1 / rule.tau), x.k[rows].double()
    else:
        a = x.low.double() + (1 - x.low.double()) * plain.sigmoid(z)
        k = 1 - a
    q = x.q[rows].double()
    q = (plain.silu(q) if rule.q_silu else q) * rule.q_scale
    S_ = torch.zeros(H, D, V, dtype=torch.float64)
    a, k, q, v, out = a.view(T, H, D), k.view(T, H, D), q.view(T, H, D), x.v[rows].double().view(T, H, V), []
    for t in range(T):
        S_ = a[t][:, :, None] * S_ + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S_, q[t]))
    o = (plain.rms(torch.stack(out), rule.eps) * x.w.double()).reshape(T, -1)
    return (o if x.gate is None else o * plain.silu(x.gate[rows].double())), S_


SHAPES = [(2, 56, 32), (3, 16, 24), (2, 128, 128), (1, 64, 128), (4, 128, 64), (3, 8, 8), (2, 40, 16), (1, 13, 7), (2, 136, 200), (2, 10, 6), (1, 200, 300), (1, 5, 259)]


@pytest.mark.parametrize("H,D,V", SHAPES)
@pytest.mark.parametrize("mode", [R.BOUNDED, R.ROOT])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_recurrence_token_by_token_and_in_runs(H, D, V, mode, dtype):
    N = 37
    rule = R.StateRule(H, D, V, mode, 1e-4, q_silu=mode == R.BOUNDED, q_scale=0.3, tau=7.0)
    x, back = operands(2 * N, H, D, V, mode, 5, dtype, gate=mode == R.ROOT)
    xd = to_dev(x, back)
    want = [plain_advance(rule, x, list(range(N))), plain_advance(rule, x, list(range(N, 2 * N)))]
    for cuts in ([(0, N)], S.singles(0, N), [(0, 5), (5, 2), (7, 30)]):
        for history in (1, 4):
            state = torch.full((3, history, H, D, V), 1e30, device=DEV)
            out = torch.zeros(2 * N, H * V + 8, dtype=dtype, device=DEV)
            for lo, n in cuts:
                rows = list(range(lo, lo + n)) + list(range(N + lo, N + lo + n))
                sub = R.Operands(*[None if t is None else t[rows] for t in (xd.q, xd.k, xd.v, xd.gate, xd.z)], xd.bias, xd.low, xd.w)
                pos, slot = ints(list(range(lo, lo + n)) * 2), ints([2] * n + [0] * n)
                runs = None if n == 1 else ints([[0, n], [n, n]])
                part = torch.zeros(2 * n, H * V + 8, dtype=dtype, device=DEV)
                R.advance(rule, sub, state, SimpleNamespace(slot=slot, pos=pos, runs=runs, prompts=[], memo={}), part[:, :H * V])
                out[rows] = part
            w = torch.cat([want[0][0], want[1][0]])
            err = (out[:, :H * V].cpu().double() - w).abs().max()
            assert float(err) < (2e-5 if dtype == F32 else 1.5e-2) * float(w.abs().max()), (cuts[:2], history, float(err))
            for s, (_, st) in ((2, want[0]), (0, want[1])):
                assert torch.allclose(state[s, N % history].cpu().double(), st, atol=1e-4 * float(st.abs().max()))


def _chunked(rule, x, back, counts, pieces, monkey_sms=None):
    """Feeds runs of the given lengths as prompt portions: pieces[r] lists a run's portions; all runs advance together."""
    xd = to_dev(x, back)
    H, D, V = rule.heads, rule.dim, rule.vdim
    state = torch.full((len(counts), 1, H, D, V), 1e30, device=DEV)
    out = torch.zeros(sum(counts), H * V + 8, dtype=BF, device=DEV)
    base = [sum(counts[:i]) for i in range(len(counts))]
    for step in range(max(len(p) for p in pieces)):
        part = [(r, *pieces[r][step]) for r in range(len(counts)) if step < len(pieces[r])]
        rows = [base[r] + t for r, lo, n in part for t in range(lo, lo + n)]
        sub_rows = torch.tensor(rows, device=DEV)
        # rows stay views of wide rows: the kernel reads them with their stride
        wide, zw = back[0].to(DEV)[sub_rows], back[1].to(DEV)[sub_rows]
        def view(t, src, ref):
            if t is None:
                return None
            off = (t.data_ptr() - ref.data_ptr()) // t.element_size()
            return src[:, off:off + t.shape[1]]
        sub = R.Operands(view(x.q, wide, back[0]), view(x.k, wide, back[0]), view(x.v, wide, back[0]), view(x.gate, wide, back[0]), view(x.z, zw, back[1]),
                         xd.bias, xd.low, xd.w)
        pos = ints([t for r, lo, n in part for t in range(lo, lo + n)])
        slot = ints([r for r, lo, n in part for _ in range(n)])
        segs, at = [], 0
        for r, lo, n in part:
            segs.append(SimpleNamespace(start=at, sequences=1, count=n, slot=r, begin=lo))
            at += n
        o = torch.zeros(len(rows), H * V + 8, dtype=BF, device=DEV)
        runs = ints([[g.start, g.count] for g in segs])
        assert R._chunked(rule, sub)
        R.advance(rule, sub, state, SimpleNamespace(slot=slot, pos=pos, runs=runs, prompts=segs, memo={}), o[:, :H * V])
        out[sub_rows] = o
    return out[:, :H * V].cpu().double(), state[:, 0].cpu().double()


@pytest.mark.parametrize("H,D,V", [(2, 56, 32), (2, 128, 128), (3, 64, 128), (2, 128, 64), (1, 8, 8), (2, 40, 24)])
@pytest.mark.parametrize("mode", [R.BOUNDED, R.ROOT])
def test_recurrence_in_chunks(H, D, V, mode):
    """One stretch and many, portions that end inside a chunk, several runs at once; decays from weak to very strong (the
    shifted gates take the form without exponents out of range)."""
    rule = R.StateRule(H, D, V, mode, 1e-4, q_silu=mode == R.BOUNDED, q_scale=0.3, tau=7.0 if D != 64 else 0.5)
    for shift, scale in ((0.0, 2.0), (8.0, 1.0), (-6.0, 3.0), (-40.0, 30.0)):
        counts = [700, 33, 130, 64]
        x, back = operands(sum(counts), H, D, V, mode, 7, BF, mode == R.ROOT, shift, scale)
        base = [sum(counts[:i]) for i in range(4)]
        want = [plain_advance(rule, x, list(range(b, b + n))) for b, n in zip(base, counts)]
        w = torch.cat([o for o, _ in want])
        for pieces in ([[(0, n)] for n in counts], [[(0, 100), (100, 33), (133, 567)], [(0, 33)], [(0, 65), (65, 65)], [(0, 32), (32, 32)]]):
            got, state = _chunked(rule, x, back, counts, pieces)
            err = (got - w).abs()
            assert float(err.max()) < 2e-2 * float(w.abs().max()), (shift, int(err.max(1).values.argmax()), float(err.max()))
            for r, (_, st) in enumerate(want):
                assert float((state[r] - st).abs().max()) < 2e-4 * max(float(st.abs().max()), 1e-3), (shift, r)


def test_stretches_of_one_run_agree_with_one_stretch(monkeypatch):
    rule = R.StateRule(2, 128, 128, R.BOUNDED, 1e-4, q_silu=True)
    x, back = operands(1500, 2, 128, 128, R.BOUNDED, 9, BF, False, 2.0, 1.0)
    want, st = plain_advance(rule, x, list(range(1500)))
    for sms in (1, 8, 148):
        monkeypatch.setattr(R, "SMS", sms)
        got, state = _chunked(rule, x, back, [1500], [[(0, 1500)]])
        assert float((got - want).abs().max()) < 2e-2 * float(want.abs().max()), sms
        assert float((state[0] - st).abs().max()) < 2e-4 * float(st.abs().max()), sms


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", ["mixed", "odd", "wide", "long_heads"])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_prompts_portions_and_decoding_match_the_restatement(name, dtype):
    d, cfg, t = S.build(name)
    n = 200
    toks = S.tokens(n, cfg.vocab_size, 1)
    want = S.expect(d, t, toks)
    e = S.engine(cfg, t, DEV, dtype)
    for cuts in ([(0, n)], S.singles(0, n), S.portions(n, [33, 2, 64, 5]), S.portions(n, [2]), S.portions(n, [100, 3]),
                 [(0, 60), (60, 32)] + S.singles(92, n)):
        S.assert_close(S.feed(e, toks, cuts), want, dtype, (name, cuts[:3]))
    eager = S.engine(cfg, t, DEV, dtype, use_graph=False)
    S.assert_close(S.feed(eager, toks, S.singles(0, n)), want, dtype, "without graphs")


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
def test_batches_of_unequal_sequences_and_pages_and_slots_used_again(dtype):
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
        for i in (2, 0, 3, 1):
            S.assert_close(torch.cat(got[i]), want[i], dtype, i)
            e.close(slots[i])


def test_long_decoding_in_both_types():
    """700 tokens, most of them decoded one by one: in fp32 one key too many or a state a token late is visible."""
    layers = [(S.attention(4, 2, 16, 16, 0.4, 300), 32), (S.hgrn2(2, 24, 16), 32), (S.gla(2, 16, 24, 8.0, 4), 32), (S.attention(4, 2, 16, 16, 0.4, 128, kv_from=0), 32)]
    d = S.config(48, 60, layers)
    cfg = S.NufalornConfig.from_dict(d)
    t = S.random_tensors(cfg, 2)
    toks = S.tokens(700, 60, 3)
    want = S.expect(d, t, toks)
    for dtype in (F32, BF):
        e = S.engine(cfg, t, DEV, dtype)
        S.assert_close(S.feed(e, toks, [(0, 90)] + S.singles(90, 700)), want, dtype)
        S.assert_close(S.feed(e, toks, S.portions(700, [129, 64, 2])), want, dtype)
        S.assert_close(S.feed(e, toks, [(0, 700)]), want, dtype)


def test_greedy_generation_through_the_scheduler_and_the_command_line(tmp_path):
    import json

    from cogito_b200.cli import main
    from cogito_b200.serve.scheduler import Scheduler
    d, cfg, t = S.build("mixed", 7)
    prompts = [S.tokens(n, cfg.vocab_size, n) for n in (5, 70, 1, 44, 12)]
    want = [S.greedy(d, t, p, 6) for p in prompts]
    e = S.engine(cfg, t, DEV, F32, slots=3, pool=320)
    s = Scheduler(e, step_tokens=48)
    reqs = [s.add(p, 6) for p in prompts]
    s.run()
    assert [r.tokens for r in reqs] == want
    assert e.free_slots() == 3 and e.cache.free_pages() == e.cache.n_pages - 1
    registry.save_folder(str(tmp_path / "m"), cfg, t)
    (tmp_path / "p.json").write_text(json.dumps(prompts))
    main(["generate", f"model.path={tmp_path}/m", "generate.dtype=float32", f"generate.prompts={tmp_path}/p.json", "generate.new_tokens=6",
          f"generate.out={tmp_path}/o.json"])
    assert json.loads((tmp_path / "o.json").read_text()) == [p + w for p, w in zip(prompts, want)]


def test_speculative_decoding_takes_back_states():
    from cogito_b200.models.nufalorn import Nufalorn
    from cogito_b200.serve.engine import SpeculativeDecoder
    from cogito_b200.serve.stack import StackEngine
    d, cfg, t = S.build("mixed", 7)
    other = S.random_tensors(cfg, 8)
    draft = Nufalorn(cfg, {k: (0.9 * v.float() + 0.1 * other[k].float()).to(v.dtype) for k, v in t.items()}, DEV, F32)
    m = Nufalorn(cfg, t, DEV, F32)
    prompts = torch.tensor([S.tokens(40, cfg.vocab_size, 1), S.tokens(40, cfg.vocab_size, 2)])
    want = [S.greedy(d, t, p.tolist(), 10) for p in prompts]
    for dr, all_accepted in ((m, True), (draft, False)):
        dec = SpeculativeDecoder(StackEngine(dr, 2, 256), StackEngine(m, 2, 256), gamma=3, temperature=0.0)
        seqs, stats = dec.generate(prompts.to(DEV), 10)
        assert (stats.acceptance_rate == 1.0) == all_accepted
        assert [s[40:50] for s in seqs] == want
        dec.close()


def test_trace_runner_program(tmp_path):
    import json
    import subprocess
    import sys
    from pathlib import Path

    import numpy as np
    d, cfg, t = S.build("wide", 2)
    registry.save_folder(str(tmp_path / "m"), cfg, t)
    toks = S.tokens(80, cfg.vocab_size, 1)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:78], "want": [0, 77]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[78:79], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[79:], "want": [0]}], "end": ["a"]}]
    root = Path(__file__).resolve().parent.parent
    want = S.expect(d, t, toks)[[0, 77, 79]]
    for dtype in ("float32", "bfloat16"):
        r = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path),
                            "--max-tokens", "96"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=200)
        assert r.returncode == 0, r.stderr
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
        got = torch.from_numpy(np.concatenate([np.fromfile(tmp_path / f"{i}.f32", dtype="<f4") for i in (0, 2)]).reshape(3, -1)).double()
        S.assert_close(got, want, getattr(torch, dtype))
