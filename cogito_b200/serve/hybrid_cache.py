"""Cache of models that mix attention layers with recurrent ones: paged keys and values for the layers that own some,
one fp32 state per sequence slot for the recurrent layers.

Keys and values: per layer ``k_pages[n_pages, kv_heads, page_size, ceil8(dim)]`` and ``v_pages`` likewise with vdim, as the
attention sees them (rotated, normed), in bf16 or fp32; a layer that reads another layer's cache has no pages of its own.
States: per layer ``[slots, history, heads, dim, vdim]``; the state after p tokens is entry p mod history, so a caller may
take back up to history - 1 tokens by setting ``lengths`` back.  A pooled cache keeps one entry.  Nothing is cleared when
a slot or a page changes hands: a sequence at position 0 starts from zeros, and no key beyond a sequence's own is seen.
"""
from __future__ import annotations

import ctypes
from ctypes import Structure, c_float, c_int32, c_int64, c_void_p
from dataclasses import dataclass

import torch

from ..ops import _lib
from ..ops import rotary
from ..ops.attention import turn_back
from .kv_cache import PagedCache

HISTORY = 16                # states kept per sequence where tokens may be taken back


class KvRowsArgs(Structure):
    """Mirror of ``cgk_kv_rows_args`` (include/cogito_kernels.h)."""

    _fields_ = [("k_pages", c_void_p), ("v_pages", c_void_p), ("page_table", c_void_p), ("slot", c_void_p), ("pos", c_void_p),
                ("kv_heads", c_int32), ("dim", c_int32), ("vdim", c_int32), ("page_size", c_int32), ("max_pages", c_int32),
                ("slots", c_int32), ("n_pages", c_int32), ("fp32", c_int32)]


class KvPrepArgs(Structure):
    """Mirror of ``cgk_kv_prep_args`` (include/cogito_kernels.h)."""

    _fields_ = [("q", c_void_p), ("k", c_void_p), ("v", c_void_p), ("ldq", c_int64), ("ldk", c_int64), ("ldv", c_int64),
                ("cs_k", c_void_p), ("cs_v", c_void_p), ("q_out", c_void_p), ("k_out", c_void_p), ("v_out", c_void_p),
                ("heads", c_int32), ("rot", c_int32), ("wide", c_int32), ("norm_v", c_int32), ("eps", c_float)]


@dataclass(frozen=True)
class KvShape:
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class StateShape:
    heads: int
    dim: int
    vdim: int


def _ceil8(n: int) -> int:
    return (n + 7) // 8 * 8


def _widen(x, wide):
    """x [.., d] -> [.., wide] with zeros after the row's own elements."""
    return torch.nn.functional.pad(x, (0, wide - x.shape[-1]))


class HybridCache(PagedCache):
    """layers: KvShape (owns keys and values), StateShape, or an int (reads that layer's keys and values), per layer."""

    def __init__(self, layers, batch: int, max_seq_len: int, page_size: int = 64, device="cpu", dtype=torch.bfloat16, n_pages: int | None = None):
        super().__init__(batch, max_seq_len, page_size, device, n_pages)
        self.dtype, self.history = dtype, 1 if self.pooled else HISTORY
        self.kv: dict[int, tuple[KvShape, torch.Tensor, torch.Tensor]] = {}
        self.states: dict[int, torch.Tensor] = {}
        for i, l in enumerate(layers):
            if isinstance(l, KvShape):
                mk = lambda d: torch.zeros(self.n_pages, l.heads, page_size, _ceil8(d), dtype=dtype, device=self.device)
                self.kv[i] = (l, mk(l.dim), mk(l.vdim))
            elif isinstance(l, StateShape):
                self.states[i] = torch.zeros(batch, self.history, l.heads, l.dim, l.vdim, dtype=torch.float32, device=self.device)
        for i, l in enumerate(layers):
            if isinstance(l, int):
                self.kv[i] = self.kv[l]

    def nbytes(self) -> int:
        own = {id(t): t for _, k, v in self.kv.values() for t in (k, v)}
        return sum(t.numel() * t.element_size() for t in [*own.values(), *self.states.values()])

    def _args(self, layer: int, slot=None, pos=None) -> KvRowsArgs:
        s, k, v = self.kv[layer]
        a = KvRowsArgs()
        a.k_pages, a.v_pages, a.page_table = k.data_ptr(), v.data_ptr(), self.page_table.data_ptr()
        a.slot, a.pos = _lib.ptr(slot), _lib.ptr(pos)
        a.kv_heads, a.dim, a.vdim, a.page_size, a.max_pages = s.heads, s.dim, s.vdim, self.page_size, self.max_pages
        a.slots, a.n_pages, a.fp32 = self.batch, self.n_pages, int(self.dtype == torch.float32)
        return a

    # ------------------------------------------------------------ keys and values
    def rotate_append(self, layer: int, q, k, v, cs_k, cs_v, heads: int, wide: int, slot, pos, norm_eps: float | None, keep: bool):
        """q [N, heads * dim], k and v [N, kv_heads * .] views of the products (k and v None: the layer reads another's).
        Queries and keys are turned by cs_k, values are RMS-normed (norm_eps not None) and turned by cs_v (if given);
        keys and values go to the tokens' places.  Returns queries [N, heads, wide] and, with ``keep``, keys and values
        [N, kv_heads, wide] (None without)."""
        s, kp, vp = self.kv[layer]
        N, G = q.shape[0], s.heads
        if not q.is_cuda:
            def spin(x, n, d, cs):
                x = x.float().reshape(N, n, d)
                return x if cs is None else rotary.turn(x, cs)
            qr = _widen(spin(q, heads, s.dim, cs_k).to(self.dtype), wide)
            if k is None:
                return qr, None, None
            kr, vr = spin(k, G, s.dim, cs_k).to(self.dtype), v.float().reshape(N, G, s.vdim)
            if norm_eps is not None:
                vr = vr * torch.rsqrt((vr * vr).mean(-1, keepdim=True) + norm_eps)
            vr = (vr if cs_v is None else rotary.turn(vr, cs_v)).to(self.dtype)
            page, off = self.page_table[slot.long(), (pos // self.page_size).long()].long(), (pos % self.page_size).long()
            kp[page, :, off, :s.dim], vp[page, :, off, :s.vdim] = kr, vr
            return qr, _widen(kr, wide) if keep else None, _widen(vr, wide) if keep else None
        mk = lambda n: torch.empty(N, n, wide, dtype=self.dtype, device=q.device)
        a = KvPrepArgs()
        qr, kr, vr = mk(heads), None, None
        a.q, a.ldq, a.q_out = q.data_ptr(), q.stride(0), qr.data_ptr()
        if cs_k is not None:
            a.cs_k, a.rot = cs_k.data_ptr(), 2 * cs_k.shape[1]
        if k is not None:
            a.k, a.v, a.ldk, a.ldv, a.cs_v = k.data_ptr(), v.data_ptr(), k.stride(0), v.stride(0), _lib.ptr(cs_v)
            if keep:
                kr, vr = mk(G), mk(G)
                a.k_out, a.v_out = kr.data_ptr(), vr.data_ptr()
        a.heads, a.wide, a.norm_v, a.eps = heads, wide, int(norm_eps is not None), float(norm_eps or 0.0)
        c = self._args(layer, slot, pos)
        _lib.check(_lib.lib().cgk_kv_rotate_append(ctypes.byref(c), ctypes.byref(a), N, _lib.stream_ptr()), "cgk_kv_rotate_append")
        _lib.count_launch()
        return qr, kr, vr

    def gather(self, layer: int, slot: int, first: int, length: int, wide: int):
        """Keys and values [length, kv_heads, wide] of positions first .. of the sequence in ``slot``."""
        s, kp, vp = self.kv[layer]
        if self.device.type != "cuda":
            pos = torch.arange(first, first + length)
            page, off = self.page_table[slot, pos // self.page_size].long(), pos % self.page_size
            return tuple(_widen(t[page, :, off, :d], wide) for t, d in ((kp, s.dim), (vp, s.vdim)))
        k, v = (torch.empty(length, s.heads, wide, dtype=self.dtype, device=self.device) for _ in range(2))
        c = self._args(layer)
        _lib.check(_lib.lib().cgk_kv_gather(ctypes.byref(c), slot, first, length, wide, k.data_ptr(), v.data_ptr(), _lib.stream_ptr()), "cgk_kv_gather")
        _lib.count_launch()
        return k, v

    ROWS = 32768                # query tokens per launch

    def attention(self, layer: int, q, slot, pos, scale: float, max_len: int, out, block: int = 0, sink: bool = False, turn=None, splits: int = 0):
        """q [N, heads, wide]; token t stands at pos[t] of the sequence in slot[t] and sees its keys 0 .. pos[t] (all appended),
        with ``block`` those of its own block of positions.  ``sink``: one is added to the softmax denominator.  The result
        goes to ``out`` [N, heads * vdim] (a view with longer rows is fine), turned back by ``turn`` [N, vdim / 2, 2].
        ``max_len`` bounds the sequence lengths (it sizes the key ranges, not the result)."""
        s, kp, vp = self.kv[layer]
        N, H, wide = q.shape
        group = H // s.heads
        if not q.is_cuda:
            for t in range(N):
                p = int(pos[t])
                lo = p // block * block if block else 0
                k, v = (x.float().repeat_interleave(group, 1) for x in self.gather(layer, int(slot[t]), lo, p + 1 - lo, max(wide, s.vdim)))
                sc = torch.einsum("hd,khd->hk", q[t].float(), k[..., :wide]) * scale
                if sink:
                    sc = torch.cat([sc, torch.zeros(H, 1)], 1)
                o = torch.einsum("hk,khd->hd", torch.softmax(sc, -1)[:, :p + 1 - lo], v[..., :s.vdim])
                out[t] = (o if turn is None else turn_back(o, turn[t])).reshape(-1).to(out.dtype)
            return out
        L = _lib.lib()
        longest = min(block, max_len) if block else max_len
        for i in range(0, N, self.ROWS):
            n = min(self.ROWS, N - i)
            if splits <= 0:
                ctas = n * s.heads * (1 if group <= 2 else (group + 3) // 4)
                splits = max(1, min(32, 1536 // ctas, (longest + 63) // 64))
            need = L.cgk_kv_rows_scratch_floats(n, H, s.vdim, splits)
            scratch = torch.empty(need, dtype=torch.float32, device=q.device) if need else None
            a = self._args(layer, slot[i:], pos[i:])
            _lib.check(L.cgk_kv_rows_attention(ctypes.byref(a), q[i:].data_ptr(), q.stride(0), wide, out[i:].data_ptr(), out.stride(0),
                                               None if turn is None else turn[i:].data_ptr(), n, H, float(scale), int(block), int(sink), splits,
                                               _lib.ptr(scratch), _lib.stream_ptr()), "cgk_kv_rows_attention")
            _lib.count_launch(2 if splits > 1 else 1)
        return out
