"""Mixture-of-experts routing and expert products.

``route`` picks each token's outputs (softmax scores, additive correction for the choice only, group-limited
selection, identity outputs); ``expert_outputs`` runs the chosen experts: grouped tcgen05 GEMMs over rows
permuted into expert order, or one warp per output element when there are few (token, choice) pairs, in
fp32, or when the sizes do not satisfy TMA's alignment.  CUDA: csrc/kernels/moe.cu and gemm_tcgen05.cu.
CPU tensors take an fp32 restatement.
"""
from __future__ import annotations

import torch

from . import _lib

FEW_PAIRS = 32           # up to here every pair reads its expert's weights by itself
TILE = 128               # row tile of the grouped GEMM


class Routing:
    """idx [N, top] int32 outputs, weight [N, top] fp32, row_of [N, top] int32 (row of the pair's result, -1: the
    output is the input itself), counts: device counters per expert (grouped path)."""

    def __init__(self, idx, weight, row_of, counts=None):
        self.idx, self.weight, self.row_of, self.counts = idx, weight, row_of, counts


_counts: dict = {}


def _counters(device, experts: int) -> torch.Tensor:
    """int32 per expert, zero between calls (the plan kernel clears what the route kernel counted)."""
    key = (device, experts)
    if key not in _counts:
        _counts[key] = torch.zeros(experts, dtype=torch.int32, device=device)
    return _counts[key]


def route(logits, correction, experts: int, top: int, groups: int = 1, keep: int = 1, count: bool = False) -> Routing:
    """logits fp32 [N, outputs]; outputs >= ``experts`` are identity outputs."""
    N, O = logits.shape
    if not logits.is_cuda:
        s = torch.softmax(logits.float(), -1)
        choice = s + correction
        if groups > 1:
            g = choice.view(N, groups, -1).amax(-1)
            best = torch.argsort(-g, dim=-1, stable=True)[:, :keep]
            allowed = torch.zeros(N, groups, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(O // groups, 1)
            choice = choice.masked_fill(~allowed, float("-inf"))
        idx = torch.argsort(-choice, dim=-1, stable=True)[:, :top]
        w = s.gather(1, idx)
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
        pair = torch.arange(N * top).view(N, top)
        return Routing(idx.to(torch.int32), w, torch.where(idx < experts, pair, torch.full_like(pair, -1)).to(torch.int32))
    dev = logits.device
    idx = torch.empty(N, top, dtype=torch.int32, device=dev)
    weight = torch.empty(N, top, dtype=torch.float32, device=dev)
    row_of = torch.empty(N, top, dtype=torch.int32, device=dev)
    counts = _counters(dev, experts) if count else None
    _lib.check(_lib.lib().cgk_moe_route(logits.data_ptr(), correction.data_ptr(), N, experts, O, top, groups, keep, idx.data_ptr(),
                                        weight.data_ptr(), row_of.data_ptr(), _lib.ptr(counts), _lib.stream_ptr()), "cgk_moe_route")
    _lib.count_launch()
    return Routing(idx, weight, row_of, counts)


def grouped_ok(h, w_gate_up, w_down) -> bool:
    """The grouped tensor-core path takes bf16 rows whose lengths are multiples of 8 elements."""
    return h.is_cuda and h.dtype == torch.bfloat16 and h.shape[-1] % 8 == 0 and w_down.shape[-1] % 8 == 0


def _grouped_gemm(a, b, out, tile_expert, tiles):
    g = _lib.GemmArgs()
    g.A, g.B, g.out = a.data_ptr(), b.data_ptr(), out.data_ptr()
    g.M, g.N, g.K, g.batch = a.shape[0], b.shape[1], a.shape[1], b.shape[0]
    g.lda, g.ldb, g.ldc = a.stride(0), b.stride(1), out.stride(0)
    g.strideB = b.stride(0)
    g.alpha, g.out_fp32 = 1.0, int(out.dtype == torch.float32)
    _lib.check(_lib.lib().cgk_gemm_grouped_bf16(g, tile_expert.data_ptr(), tiles.data_ptr(), _lib.stream_ptr()), "cgk_gemm_grouped_bf16")
    _lib.count_launch()
    return out


def expert_outputs(h, r: Routing, w_gate_up, w_down):
    """h [N, D]; w_gate_up [E, 2F, D] (gate rows, then up rows), w_down [E, D, F].  Returns the rows that
    ``r.row_of`` names: W_down (silu(W_gate h) * (W_up h)) of each pair's expert."""
    N, D = h.shape
    E, F, top = w_down.shape[0], w_down.shape[2], r.idx.shape[1]
    if not h.is_cuda:
        out = torch.zeros(N * top, D)
        flat = r.idx.reshape(-1)
        for e in range(E):
            p = (flat == e).nonzero().view(-1)
            if len(p):
                gu = h[p // top].float() @ w_gate_up[e].float().T
                out[p] = (torch.nn.functional.silu(gu[:, :F]) * gu[:, F:]) @ w_down[e].float().T
        return out
    L, dev, pairs, st = _lib.lib(), h.device, N * top, _lib.stream_ptr()
    if r.counts is None:
        act = torch.empty(pairs, F, dtype=h.dtype, device=dev)
        y = torch.empty(pairs, D, dtype=torch.float32, device=dev)
        _lib.check(L.cgk_expert_rows(int(h.dtype == torch.float32), h.data_ptr(), r.idx.data_ptr(), pairs, top, E, w_gate_up.data_ptr(),
                                     w_down.data_ptr(), act.data_ptr(), y.data_ptr(), D, F, st), "cgk_expert_rows")
        _lib.count_launch(2)
        return y
    max_tiles = pairs // TILE + min(E, pairs)            # full tiles plus one started tile per expert in use
    ints = torch.empty(E + max_tiles + 1, dtype=torch.int32, device=dev)
    cursor, tile_expert, tiles = ints[:E], ints[E:E + max_tiles], ints[E + max_tiles:]
    _lib.check(L.cgk_moe_plan(r.counts.data_ptr(), E, cursor.data_ptr(), tile_expert.data_ptr(), tiles.data_ptr(), max_tiles, st), "cgk_moe_plan")
    rows = max_tiles * TILE
    xp = torch.empty(rows, D, dtype=h.dtype, device=dev)
    _lib.check(L.cgk_moe_gather(h.data_ptr(), r.idx.data_ptr(), pairs, top, E, cursor.data_ptr(), r.row_of.data_ptr(), xp.data_ptr(), D, rows, st),
               "cgk_moe_gather")
    gu = _grouped_gemm(xp, w_gate_up, torch.empty(rows, 2 * F, dtype=h.dtype, device=dev), tile_expert, tiles)
    act = torch.empty(rows, F, dtype=h.dtype, device=dev)
    _lib.check(L.cgk_swiglu_tiles(gu.data_ptr(), act.data_ptr(), tiles.data_ptr(), F, max_tiles, st), "cgk_swiglu_tiles")
    _lib.count_launch(3)
    return _grouped_gemm(act, w_down, torch.empty(rows, D, dtype=h.dtype, device=dev), tile_expert, tiles)
