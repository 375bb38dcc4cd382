"""Paged caches of the serving engines and attention over them: INT4 keys / values, and latents.

``PagedCache`` holds what both share: the page table, sequence slots and lengths.

INT4 (``PagedKVCacheInt4``): per layer the pool is ``pages[num_pages, page_size, heads, D/2]`` bytes plus fp32 scales
``[num_pages, page_size, heads, D/group]`` (one token's bytes equal the reference layout
``[layers, max_seq, heads, head_dim/2]`` of cg_kv_cache_int4, src/quantize/int4.c:116-145; a
single page of ``max_seq`` tokens reproduces it exactly).  ``lengths`` counts committed tokens
per sequence once, whatever the number of layers (the reference advances it on every
append, src/quantize/int4.c:233).  Rejected speculative tokens are dropped by not advancing
``lengths`` past them.

Latents (``PagedLatentCache``): per layer ``pages[num_pages, page_size, rank]`` in bf16 or fp32, one short row
per token from which every head's key and value follow (csrc/kernels/latent_kv.cu, latent_attn_tc.cu).
"""
from __future__ import annotations

import ctypes
import math
from ctypes import Structure, c_float, c_int32, c_void_p

import torch

from ..ops import _lib
from ..quant.int4 import _round_half_away


class KvArgs(Structure):
    _fields_ = [("k_pages", c_void_p), ("v_pages", c_void_p), ("k_scales", c_void_p), ("v_scales", c_void_p),
                ("page_table", c_void_p), ("lengths", c_void_p),
                ("batch", c_int32), ("heads", c_int32), ("D", c_int32), ("group", c_int32),
                ("page_size", c_int32), ("max_pages", c_int32)]


class PagedCache:
    """Page table, sequence slots and committed lengths, whatever a page holds.

    ``n_pages=None``: identity placement, slot b owns pages b * max_pages .. (a fixed batch of sequences; any
    permutation of ``page_table`` works).  Otherwise the pool has ``n_pages`` pages and a sequence takes them as
    it grows: ``open`` a slot, ``reserve`` room before a step, ``close`` it and its pages serve other sequences."""

    def __init__(self, batch: int, max_seq_len: int, page_size: int, device="cpu", n_pages: int | None = None):
        self.batch, self.page_size = batch, page_size
        self.max_pages = (max_seq_len + page_size - 1) // page_size
        self.device = torch.device(device)
        self.pooled = n_pages is not None
        self.n_pages = n_pages if self.pooled else batch * self.max_pages
        self.lengths = torch.zeros(batch, dtype=torch.int32, device=self.device)
        if self.pooled:
            self.page_table = torch.zeros(batch, self.max_pages, dtype=torch.int32, device=self.device)
            self._free_pages = list(range(self.n_pages - 1, -1, -1))
            self._free_slots = list(range(batch - 1, -1, -1))
            self._owned: dict[int, list[int]] = {}
        else:
            self.page_table = torch.arange(self.n_pages, dtype=torch.int32, device=self.device).view(batch, self.max_pages)

    def reset(self):
        self.lengths.zero_()
        if self.pooled:
            for slot in list(self._owned):
                self.close(slot)

    def commit(self, n_tokens):
        """Advance the lengths (int or per-sequence tensor) after the appended tokens are accepted."""
        self.lengths += n_tokens

    # ------------------------------------------------------- slots and pages of a pooled cache
    def open(self) -> int:
        """Takes a free sequence slot."""
        if not self._free_slots:
            raise RuntimeError("no free sequence slot")
        slot = self._free_slots.pop()
        self._owned[slot] = []
        return slot

    def free_slots(self) -> int:
        return len(self._free_slots)

    def free_pages(self) -> int:
        return len(self._free_pages)

    def pages_for(self, length: int) -> int:
        return (length + self.page_size - 1) // self.page_size

    def reserve(self, slot: int, length: int):
        """Gives the sequence in ``slot`` the pages that ``length`` tokens need."""
        own = self._owned[slot]
        need = self.pages_for(length)
        if need <= len(own):
            return
        if need > self.max_pages:
            raise ValueError(f"a sequence of {length} tokens exceeds the cache's {self.max_pages * self.page_size}")
        if need - len(own) > len(self._free_pages):
            raise RuntimeError(f"the page pool is exhausted: {need - len(own)} pages wanted, {len(self._free_pages)} free")
        first = len(own)
        own.extend(self._free_pages.pop() for _ in range(need - first))
        self.page_table[slot, first:need] = torch.tensor(own[first:], dtype=torch.int32).to(self.device)

    def close(self, slot: int):
        """Returns the slot and its pages."""
        self._free_pages.extend(reversed(self._owned.pop(slot)))
        self._free_slots.append(slot)


class PagedKVCacheInt4(PagedCache):
    def __init__(self, num_layers: int, batch: int, max_seq_len: int, heads: int, head_dim: int, group: int = 32,
                 page_size: int = 64, device="cpu"):
        if head_dim % group or group % 8:
            raise ValueError("group must be a multiple of 8 that divides head_dim")
        super().__init__(batch, max_seq_len, page_size, device)
        self.num_layers, self.heads, self.D, self.group = num_layers, heads, head_dim, group
        n_pages = self.n_pages
        G = head_dim // group
        mk = lambda *s, dt: torch.zeros(*s, dtype=dt, device=self.device)
        self.k_pages = [mk(n_pages, page_size, heads, head_dim // 2, dt=torch.uint8) for _ in range(num_layers)]
        self.v_pages = [mk(n_pages, page_size, heads, head_dim // 2, dt=torch.uint8) for _ in range(num_layers)]
        self.k_scales = [mk(n_pages, page_size, heads, G, dt=torch.float32) for _ in range(num_layers)]
        self.v_scales = [mk(n_pages, page_size, heads, G, dt=torch.float32) for _ in range(num_layers)]
        self._scratch = None

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for ts in (self.k_pages, self.v_pages, self.k_scales, self.v_scales) for t in ts)

    def _args(self, layer: int) -> KvArgs:
        a = KvArgs()
        a.k_pages, a.v_pages = self.k_pages[layer].data_ptr(), self.v_pages[layer].data_ptr()
        a.k_scales, a.v_scales = self.k_scales[layer].data_ptr(), self.v_scales[layer].data_ptr()
        a.page_table, a.lengths = self.page_table.data_ptr(), self.lengths.data_ptr()
        a.batch, a.heads, a.D, a.group = self.batch, self.heads, self.D, self.group
        a.page_size, a.max_pages = self.page_size, self.max_pages
        return a

    # ------------------------------------------------------------------ append
    def append(self, layer: int, k_new: torch.Tensor, v_new: torch.Tensor):
        """k_new, v_new: [batch, T, heads, D]; stored at positions lengths[b] .. lengths[b]+T-1."""
        B, T, H, D = k_new.shape
        if (B, H, D) != (self.batch, self.heads, self.D):
            raise ValueError("shape does not match the cache")
        if k_new.is_cuda:
            k_new, v_new = k_new.to(torch.bfloat16).contiguous(), v_new.to(torch.bfloat16).contiguous()
            a = self._args(layer)
            _lib.check(_lib.lib().cgk_kv_int4_append(ctypes.byref(a), k_new.data_ptr(), v_new.data_ptr(), T,
                                                     _lib.stream_ptr()), "cgk_kv_int4_append")
            _lib.count_launch()
            return
        G = D // self.group
        for src, pages, scales in ((k_new, self.k_pages[layer], self.k_scales[layer]), (v_new, self.v_pages[layer], self.v_scales[layer])):
            x = src.to(torch.bfloat16).float().view(B, T, H, G, self.group)
            amax = x.abs().amax(-1)
            s = torch.where(amax < 1e-10, torch.ones_like(amax), amax / 7.0)
            q = _round_half_away(x / s[..., None]).clamp_(-8, 7).to(torch.int16).view(B, T, H, D) & 0xF
            packed = (q[..., 0::2] | (q[..., 1::2] << 4)).to(torch.uint8)
            for b in range(B):
                for t in range(T):
                    pos = int(self.lengths[b]) + t
                    page = int(self.page_table[b, pos // self.page_size])
                    pages[page, pos % self.page_size] = packed[b, t]
                    scales[page, pos % self.page_size] = s[b, t]

    # -------------------------------------------------------------------- read
    def gather(self, layer: int, b: int, length: int):
        """Dequantised (k, v) [length, heads, D] of one sequence (fp32)."""
        out = []
        for pages, scales in ((self.k_pages[layer], self.k_scales[layer]), (self.v_pages[layer], self.v_scales[layer])):
            pos = torch.arange(length, device=self.device)
            page = self.page_table[b, (pos // self.page_size).long()].long()
            raw = pages[page, (pos % self.page_size).long()].to(torch.int16)          # [len, H, D/2]
            q = torch.stack([raw & 0xF, raw >> 4], -1).reshape(length, self.heads, self.D)
            q = torch.where(q >= 8, q - 16, q).float()
            s = scales[page, (pos % self.page_size).long()]                          # [len, H, G]
            out.append(q * s.repeat_interleave(self.group, -1))
        return out

    def attention(self, layer: int, q: torch.Tensor, splits: int = 0) -> torch.Tensor:
        """q: [batch, Tq, Hq, D], the Tq newest tokens (already appended, not yet committed).
        Query t sees keys 0 .. lengths[b] + t."""
        B, Tq, Hq, D = q.shape
        scale = 1.0 / math.sqrt(D)
        if q.is_cuda:
            q = q.to(torch.bfloat16).contiguous()
            if splits <= 0:
                longest = self.max_pages * self.page_size
                splits = max(1, min(32, 296 // max(1, B * self.heads), (longest + 255) // 256))
            L = _lib.lib()
            need = L.cgk_kv_int4_attention_scratch_floats(B, Hq, Tq, D, splits)
            if self._scratch is None or self._scratch.numel() < need:
                self._scratch = torch.empty(need, dtype=torch.float32, device=q.device)
            out = torch.empty_like(q)
            a = self._args(layer)
            _lib.check(L.cgk_kv_int4_attention(ctypes.byref(a), q.data_ptr(), out.data_ptr(), Tq, Hq, scale, splits,
                                               self._scratch.data_ptr(), _lib.stream_ptr()), "cgk_kv_int4_attention")
            _lib.count_launch(2)
            return out
        out = torch.empty(B, Tq, Hq, D, dtype=q.dtype)
        rep = Hq // self.heads
        for b in range(B):
            n = int(self.lengths[b]) + Tq
            k, v = self.gather(layer, b, n)
            k, v = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
            s = torch.einsum("qhd,khd->hqk", q[b].to(torch.bfloat16).float(), k) * scale
            mask = torch.arange(n)[None, :] > (torch.arange(Tq)[:, None] + n - Tq)
            s = s.masked_fill(mask[None], float("-inf"))
            out[b] = torch.einsum("hqk,khd->qhd", torch.softmax(s, -1), v).to(q.dtype)
        return out


class LatentArgs(Structure):
    """Mirror of ``cgk_latent_args`` (include/cogito_kernels.h)."""

    _fields_ = [("pages", c_void_p), ("page_table", c_void_p), ("slot", c_void_p), ("pos", c_void_p),
                ("R", c_int32), ("page_size", c_int32), ("max_pages", c_int32), ("slots", c_int32), ("n_pages", c_int32),
                ("heads", c_int32), ("fp32", c_int32), ("scale", c_float)]


class PagedLatentCache(PagedCache):
    """``ranks``: latent size of every layer run (layers may differ).  Pages start as zeros and only ever receive
    finite rows: the tensor-core kernel reads whole pages and gives keys beyond the sequence the weight 0."""

    def __init__(self, ranks, batch: int, max_seq_len: int, page_size: int = 64, device="cpu", dtype=torch.bfloat16, n_pages: int | None = None):
        super().__init__(batch, max_seq_len, page_size, device, n_pages)
        self.ranks, self.dtype = list(ranks), dtype
        self.pages = [torch.zeros(self.n_pages, page_size, r, dtype=dtype, device=self.device) for r in self.ranks]

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.pages)

    def _args(self, layer: int, slot=None, pos=None, heads: int = 0, scale: float = 1.0) -> LatentArgs:
        a = LatentArgs()
        a.pages, a.page_table = self.pages[layer].data_ptr(), self.page_table.data_ptr()
        # the struct's users check for null; the gather does not look at slot and pos
        a.slot, a.pos = _lib.ptr(slot), _lib.ptr(pos)
        a.R, a.page_size, a.max_pages, a.slots, a.n_pages = self.ranks[layer], self.page_size, self.max_pages, self.batch, self.n_pages
        a.heads, a.fp32, a.scale = heads, int(self.dtype == torch.float32), float(scale)
        return a

    def _place(self, slot, pos):
        page = self.page_table[slot.long(), (pos // self.page_size).long()].long()
        return page, (pos % self.page_size).long()

    def norm_append(self, layer: int, lat, wq, wc, eps: float, slot, pos, keep: bool):
        """lat [N, q_rank + rank] (the two down-projections side by side) -> the RMS-normed query latents [N, q_rank];
        the RMS-normed key/value latents go to their cache places (and come back as well with ``keep``)."""
        qr, R, N = wq.shape[0], self.ranks[layer], lat.shape[0]
        if not lat.is_cuda:
            def norm(v, w):
                v = v.float()
                return (v * torch.rsqrt((v * v).mean(-1, keepdim=True) + eps) * w).to(self.dtype)
            c = norm(lat[:, qr:], wc)
            page, off = self._place(slot, pos)
            self.pages[layer][page, off] = c
            return norm(lat[:, :qr], wq), c
        cq = torch.empty(N, qr, dtype=self.dtype, device=lat.device)
        c = torch.empty(N, R, dtype=self.dtype, device=lat.device) if keep else None
        a = self._args(layer, slot, pos)
        _lib.check(_lib.lib().cgk_latent_norm_append(ctypes.byref(a), lat.data_ptr(), int(lat.dtype == torch.float32), lat.stride(0), wq.data_ptr(),
                                                     wc.data_ptr(), qr, float(eps), cq.data_ptr(), _lib.ptr(c), N, _lib.stream_ptr()),
                   "cgk_latent_norm_append")
        _lib.count_launch()
        return cq, c

    def gather(self, layer: int, slot: int, length: int) -> torch.Tensor:
        """The first ``length`` latents of the sequence in ``slot``, contiguous."""
        if self.device.type != "cuda":
            pos = torch.arange(length)
            page, off = self._place(torch.full_like(pos, slot), pos)
            return self.pages[layer][page, off]
        out = torch.empty(length, self.ranks[layer], dtype=self.dtype, device=self.device)
        a = self._args(layer)
        _lib.check(_lib.lib().cgk_latent_gather(ctypes.byref(a), slot, length, out.data_ptr(), _lib.stream_ptr()), "cgk_latent_gather")
        _lib.count_launch()
        return out

    def attention(self, layer: int, q, slot, pos, scale: float, max_len: int, force_simt: bool = False) -> torch.Tensor:
        """q [N, H, rank], queries mapped into the latent space; token t stands at pos[t] of the sequence in slot[t]
        and sees its latents 0 .. pos[t] (all appended).  Returns softmax(scale q c^T) c.  ``max_len`` bounds the
        sequence lengths (it sizes the key ranges, not the result)."""
        N, H, R = q.shape
        if not q.is_cuda:
            out = torch.empty(N, H, R, dtype=q.dtype)
            for t in range(N):
                c = self.gather(layer, int(slot[t]), int(pos[t]) + 1).float()
                out[t] = (torch.softmax(q[t].float() @ c.T * scale, -1) @ c).to(q.dtype)
            return out
        L = _lib.lib()
        out = torch.empty_like(q)
        splits = 1
        if q.dtype == torch.bfloat16 and not force_simt and L.cgk_latent_attention_tc_ok(R, self.page_size, H):
            # CTAs per key range: one per token and group of up to 32 heads; ranges of whole 128-key blocks
            groups = (H + 31) // 32
            splits = max(1, min(32, 148 // max(1, N * groups), (max_len + 127) // 128))
        need = L.cgk_latent_attention_scratch_floats(N, H, R, splits)
        scratch = torch.empty(need, dtype=torch.float32, device=q.device) if need else None
        a = self._args(layer, slot, pos, H, scale)
        _lib.check(L.cgk_latent_attention(ctypes.byref(a), q.data_ptr(), out.data_ptr(), N, splits, _lib.ptr(scratch), int(force_simt),
                                          _lib.stream_ptr()), "cgk_latent_attention")
        _lib.count_launch(2 if splits > 1 else 1)
        return out
