"""Linear recurrences with a decay per state row, token by token within each sequence:

    S <- diag(a) S + k v^T,   o = S^T q     per head;   result rms(o) * w, optionally times silu(gate)

The decay comes from y = z + bias in one of two ways: ``bounded`` a = low + (1 - low) sigmoid(y) with k = 1 - a, or
``root`` a = sigmoid(y)^(1 / tau) with k given.  States, decays and everything between are fp32; q, k, v, gate and the
result have the operands' type.  CUDA: csrc/kernels/linear_state.cu (token by token: decoding, short portions, fp32)
and linear_state_tc.cu (prompt portions in chunks on the tensor cores).  CPU tensors take an fp32 restatement.
"""
from __future__ import annotations

import ctypes
from ctypes import Structure, c_float, c_int32, c_int64, c_void_p
from dataclasses import dataclass

import torch

from . import _lib

BOUNDED, ROOT = 0, 1


class LinearStateArgs(Structure):
    """Mirror of ``cgk_linear_state_args`` (include/cogito_kernels.h)."""

    _fields_ = [("q", c_void_p), ("k", c_void_p), ("v", c_void_p), ("gate", c_void_p), ("z", c_void_p),
                ("ldq", c_int64), ("ldk", c_int64), ("ldv", c_int64), ("ldg", c_int64), ("ldz", c_int64),
                ("bias", c_void_p), ("low", c_void_p), ("w", c_void_p), ("state", c_void_p), ("out", c_void_p), ("ldo", c_int64),
                ("slot", c_void_p), ("pos", c_void_p), ("runs", c_void_p),
                ("heads", c_int32), ("D", c_int32), ("V", c_int32), ("history", c_int32), ("slots", c_int32), ("mode", c_int32),
                ("q_silu", c_int32), ("fp32", c_int32), ("q_scale", c_float), ("inv_tau", c_float), ("eps", c_float)]


@dataclass(frozen=True)
class StateRule:
    """What does not change between the calls of a layer."""
    heads: int
    dim: int
    vdim: int
    mode: int
    eps: float
    q_silu: bool = False
    q_scale: float = 1.0
    tau: float = 1.0


@dataclass
class Operands:
    """Rows of a step: q, k, v, gate [N, heads * .] views (k None with BOUNDED, gate may be None), z fp32 [N, heads * dim];
    bias, low, w fp32 vectors of the layer."""
    q: torch.Tensor
    k: torch.Tensor | None
    v: torch.Tensor
    gate: torch.Tensor | None
    z: torch.Tensor
    bias: torch.Tensor
    low: torch.Tensor | None
    w: torch.Tensor


def decay_and_key(rule: StateRule, x: Operands):
    """fp32 (a, k), each [N, heads, dim]."""
    shape = (x.z.shape[0], rule.heads, rule.dim)
    y = x.z.float() + x.bias
    if rule.mode == ROOT:
        return torch.exp(torch.nn.functional.logsigmoid(y) / rule.tau).view(shape), x.k.float().reshape(shape)
    a = x.low + (1 - x.low) * torch.sigmoid(y)
    return a.view(shape), ((1 - x.low) * torch.sigmoid(-y)).view(shape)


def _advance_cpu(rule, x, state, slot, pos, runs, out):
    H, D, V, hist = rule.heads, rule.dim, rule.vdim, state.shape[1]
    a, k = decay_and_key(rule, x)
    q = x.q.float().reshape(-1, H, D)
    q = (torch.nn.functional.silu(q) if rule.q_silu else q) * rule.q_scale
    v = x.v.float().reshape(-1, H, V)
    for lo, n in (runs.tolist() if runs is not None else [(t, 1) for t in range(q.shape[0])]):
        s, p = int(slot[lo]), int(pos[lo])
        S = torch.zeros(H, D, V) if p == 0 else state[s, p % hist].clone()
        for t in range(lo, lo + n):
            S = a[t, :, :, None] * S + k[t, :, :, None] * v[t, :, None, :]
            o = torch.einsum("hdv,hd->hv", S, q[t])
            o = o * torch.rsqrt((o * o).mean(-1, keepdim=True) + rule.eps) * x.w
            if x.gate is not None:
                o = o * torch.nn.functional.silu(x.gate[t].float()).view(H, V)
            out[t] = o.reshape(-1).to(out.dtype)
            state[s, (p + 1 + t - lo) % hist] = S
    return out


def _args(rule, x, state, slot, pos, runs, out) -> LinearStateArgs:
    a = LinearStateArgs()
    a.q, a.ldq, a.v, a.ldv, a.z, a.ldz = x.q.data_ptr(), x.q.stride(0), x.v.data_ptr(), x.v.stride(0), x.z.data_ptr(), x.z.stride(0)
    if x.k is not None:
        a.k, a.ldk = x.k.data_ptr(), x.k.stride(0)
    if x.gate is not None:
        a.gate, a.ldg = x.gate.data_ptr(), x.gate.stride(0)
    a.bias, a.low, a.w = x.bias.data_ptr(), _lib.ptr(x.low), x.w.data_ptr()
    a.state, a.out, a.ldo = state.data_ptr(), out.data_ptr(), out.stride(0)
    a.slot, a.pos, a.runs = slot.data_ptr(), pos.data_ptr(), _lib.ptr(runs)
    a.heads, a.D, a.V, a.history, a.slots = rule.heads, rule.dim, rule.vdim, state.shape[1], state.shape[0]
    a.mode, a.q_silu, a.fp32 = rule.mode, int(rule.q_silu), int(x.q.dtype == torch.float32)
    a.q_scale, a.inv_tau, a.eps = rule.q_scale, 1.0 / rule.tau, rule.eps
    return a


CHUNK = 64                  # tokens per step of the tensor-core form
SMS = 148


def stretches(counts: list[int], heads: int, first_rows: list[int]):
    """Cuts runs of the given lengths into stretches that are handled side by side, whole chunks long.  The cut costs the
    least time by this count: rounds of CTAs (one per stretch and head) times the stretch's chunks and one more for a
    CTA's start and end; summing the stretches up, needed if any run is cut, takes about 0.4 of that again.
    Returns (items [n][4], run_items [runs][2], whether a run is cut)."""
    chunks = [-(-n // CHUNK) for n in counts]
    best = None
    for n in range(1, 33):
        length = -(-max(chunks) // n)
        items = sum(-(-c // length) for c in chunks)
        cost = -(-items * heads // SMS) * (length + 1) * (1.0 if items == len(chunks) else 1.4)
        if best is None or cost < best[0]:
            best = cost, length
    size, items, run_items = best[1] * CHUNK, [], []
    for r, (n, row) in enumerate(zip(counts, first_rows)):
        run_items.append([len(items), -(-n // size)])
        for at in range(0, n, size):
            items.append([row + at, min(size, n - at), r, int(at + size >= n)])
    return items, run_items, len(items) > len(counts)


def _chunked(rule: StateRule, x: Operands) -> bool:
    """Whether the tensor-core form takes these operands."""
    if x.q.dtype != torch.bfloat16 or not _lib.lib().cgk_linear_chunks_ok(rule.dim, rule.vdim):
        return False
    return all(t is None or (t.data_ptr() % 16 == 0 and t.stride(0) % 8 == 0) for t in (x.q, x.k, x.v, x.gate, x.z))


def _advance_chunks(a: LinearStateArgs, rule: StateRule, batch, rows: int, device):
    key = ("stretches", rule.heads)
    if key not in batch.memo:
        first = [g.start + i * g.count for g in batch.prompts for i in range(g.sequences)]
        items, run_items, cut = stretches([g.count for g in batch.prompts for _ in range(g.sequences)], rule.heads, first)
        flat = torch.tensor([v for t in items + run_items for v in t], dtype=torch.int32).to(device)
        batch.memo[key] = flat, len(items), len(run_items), cut
    flat, n, runs, cut = batch.memo[key]
    L, scratch = _lib.lib(), None
    if cut:
        scratch = torch.empty(L.cgk_linear_chunks_scratch_floats(n, rule.heads, rule.dim, rule.vdim), dtype=torch.float32, device=device)
    _lib.check(L.cgk_linear_chunks(ctypes.byref(a), rows, flat.data_ptr(), n, flat[4 * n:].data_ptr(), runs, _lib.ptr(scratch), _lib.stream_ptr()),
               "cgk_linear_chunks")
    _lib.count_launch(3 if cut else 1)


def advance(rule: StateRule, x: Operands, state, batch, out):
    """The recurrence over the runs of ``batch`` (slot, pos; runs int32 [n, 2]: first row and number of consecutive tokens of
    one sequence, None: every row is a run; prompts: the runs that come first and take the chunked form).  state fp32
    [slots, history, heads, dim, vdim]: the state after p tokens of a sequence is entry p mod history of its slot; a
    sequence at position 0 starts from zeros.  ``out`` [N, heads * vdim] may be a view with longer rows; returned."""
    slot, pos, runs = batch.slot, batch.pos, batch.runs
    if not x.q.is_cuda:
        return _advance_cpu(rule, x, state, slot, pos, runs, out)
    if batch.prompts and _chunked(rule, x) and out.data_ptr() % 16 == 0 and out.stride(0) % 8 == 0:
        _advance_chunks(_args(rule, x, state, slot, pos, None, out), rule, batch, x.q.shape[0], out.device)
        runs = runs[sum(g.sequences for g in batch.prompts):]
    n = x.q.shape[0] if runs is None else runs.shape[0]
    if n:
        a = _args(rule, x, state, slot, pos, runs, out)
        _lib.check(_lib.lib().cgk_linear_state(ctypes.byref(a), n, _lib.stream_ptr()), "cgk_linear_state")
        _lib.count_launch()
    return out
