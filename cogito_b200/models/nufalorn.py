"""Nufalorn: a decoder-only language model whose layers run a mixer and a feed-forward side by side on one residual
stream.  Mixers: attention inside blocks of positions (grouped queries, interleaved rotary positions, RMS-normed values
that turn with their position, a softmax with a sink; a layer may use another layer's keys and values), HGRN2, and gated
linear attention.  Norm weights are stored around zero, logits are soft-capped.

    x = E[tok];   x <- x + m (mixer(n1(x)) + ff(n2(x)));   logits = cap tanh(head n_final(x) / cap)

The stream x, states, scores and decays are fp32; matrix products take bf16 operands (or fp32 throughout with
``dtype=torch.float32``).  Built from the mechanisms in ``nn.block_attention``, ``nn.linear_attention``,
``nn.parallel_layer`` and ``ops.stream``; run by ``serve.stack.StackEngine``, which owns cache, batches and logits.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field

import torch
from torch import nn

from ..nn.block_attention import AttentionSpec, BlockAttention
from ..nn.latent_attention import _frozen
from ..nn.linear_attention import GatedLinearAttention, Hgrn2, RecurrentSpec
from ..nn.moe import DenseSpec, GatedMLP
from ..nn.parallel_layer import ParallelLayer
from ..ops import stream as S
from ..ops.linear import linear
from ..serve.hybrid_cache import HybridCache, KvShape, StateShape

RECURRENT = {"hgrn2": Hgrn2, "gla": GatedLinearAttention}


@dataclass(frozen=True)
class LayerSpec:
    kind: str                                   # attention, hgrn2 or gla
    mixer: AttentionSpec | RecurrentSpec
    mlp: DenseSpec | None
    a_rank: int = 0                             # gla: inner size of the decay's product (a checkpoint's tensors give it)


@dataclass(frozen=True)
class NufalornConfig:
    vocab_size: int
    width: int
    layers: tuple[LayerSpec, ...] = field(default_factory=tuple)
    residual_mult: float = 1.0
    logit_softcap: float = 30.0
    norm_eps: float = 1e-6

    architecture = "Nufalorn"

    @classmethod
    def from_dict(cls, d: dict, shapes: dict[str, tuple[int, ...]] | None = None) -> "NufalornConfig":
        """shapes: the checkpoint's tensors; they give the inner size of the gated decay (or the mixer's key ``a_rank``)."""
        layers = []
        for i, e in enumerate(d["layers"]):
            m, mlp, kind, rank = e["mixer"], e.get("mlp"), e["type"], 0
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            if kind == "attention":
                mixer = cls._attention(i, m, layers)
            elif kind in RECURRENT:
                mixer = RecurrentSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]) if kind == "gla" else 1.0)
                if kind == "gla":
                    rank = int(shapes[f"l{i}.mix.a1"][0]) if shapes and f"l{i}.mix.a1" in shapes else int(m["a_rank"])
            else:
                raise ValueError(f"layer {i}: unknown mixer {kind!r}")
            layers.append(LayerSpec(kind, mixer, None if mlp is None else DenseSpec(int(mlp["ff"])), rank))
        return cls(int(d["vocab"]), int(d["width"]), tuple(layers), float(d["residual_mult"]), float(d["logit_softcap"]), float(d["norm"]["eps"]))

    @staticmethod
    def _attention(i, m, before) -> AttentionSpec:
        rot, mask = m.get("rot"), m.get("mask")
        s = AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                          float(rot["base"]) if rot else 1.0, int(rot["dims"]) if rot else 0, int(mask["size"]) if mask else 0,
                          sink=True, norm_values=True, turn_values=bool(rot), kv_from=m.get("kv_from"))
        if s.heads % s.kv_heads:
            raise ValueError(f"layer {i}: {s.heads} query heads do not divide into {s.kv_heads} groups")
        if s.rot_dims % 2 or s.rot_dims > s.dim or (s.turn_values and s.vdim % 2):
            raise ValueError(f"layer {i}: rotated sizes must be even and fit the head")
        if s.kv_from is not None:
            j = s.kv_from
            o = before[j].mixer if 0 <= j < i and before[j].kind == "attention" else None
            if o is None or o.kv_from is not None or (o.kv_heads, o.dim, o.vdim) != (s.kv_heads, s.dim, s.vdim):
                raise ValueError(f"layer {i}: layer {j} has no keys and values that it can use")
        return s

    def to_dict(self) -> dict:
        out = []
        for l in self.layers:
            m = {k: getattr(l.mixer, k) for k in ("heads", "dim", "vdim")}
            if l.kind == "attention":
                s = l.mixer
                m.update(kv_heads=s.kv_heads, scale=s.scale)
                if s.turn_values:
                    m["rot"] = {"base": s.rot_base, "dims": s.rot_dims}
                if s.block:
                    m["mask"] = {"size": s.block}
                if s.kv_from is not None:
                    m["kv_from"] = s.kv_from
            elif l.kind == "gla":
                m.update(tau=l.mixer.tau, a_rank=l.a_rank)
            out.append({"type": l.kind, "mixer": m, "mlp": None if l.mlp is None else {"kind": "dense", "ff": l.mlp.ff}})
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width, "residual_mult": self.residual_mult,
                "logit_softcap": self.logit_softcap, "norm": {"eps": self.norm_eps}, "layers": out}

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Names and shapes of a checkpoint, linear weights [out, in]."""
        W, out = self.width, {"embed": (self.vocab_size, self.width)}
        for i, l in enumerate(self.layers):
            p, s = f"l{i}.mix.", l.mixer
            qk, v = s.heads * s.dim, s.heads * s.vdim
            out[f"l{i}.norm1"], out[p + "q"], out[p + "o"] = (W,), (qk, W), (W, v)
            if l.kind == "attention":
                if s.kv_from is None:
                    out[p + "k"], out[p + "v"] = (s.kv_heads * s.dim, W), (s.kv_heads * s.vdim, W)
            else:
                out[p + "v"], out[p + "norm"] = (v, W), (s.vdim,)
                if l.kind == "gla":
                    out.update({p + "k": (qk, W), p + "g": (v, W), p + "a1": (l.a_rank, W), p + "a2": (qk, l.a_rank), p + "a2.b": (qk,)})
                else:
                    out.update({p + "f": (qk, W), p + "f.b": (qk,), p + "lower": (qk,)})
            if l.mlp is not None:
                ff, p = l.mlp.ff, f"l{i}.mlp."
                out[f"l{i}.norm2"], out[p + "gate"], out[p + "up"], out[p + "down"] = (W,), (ff, W), (ff, W), (W, ff)
        out["final.norm"], out["head"] = (W,), (self.vocab_size, W)
        return out


def random_tensors(cfg: NufalornConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """bf16 checkpoint tensors: matrices N(0, 1 / in), stored norm weights around 0 (a mixer's around 1), lower bounds in
    [0, 0.9), gate biases that let some channels remember for long."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        t = torch.randn(shape, generator=g, device=device)
        if name.endswith("mix.norm"):
            t = 1.0 + 0.2 * t
        elif name.endswith("lower"):
            t = 0.9 * torch.rand(shape, generator=g, device=device)
        elif name.endswith(".b"):
            t = 2.0 + 2.0 * t
        elif len(shape) == 1:
            t = 0.2 * t
        elif name != "embed":
            t = t * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


class Nufalorn(nn.Module):
    def __init__(self, cfg: NufalornConfig, tensors: dict[str, torch.Tensor] | None = None, device="cpu", dtype=torch.bfloat16):
        """tensors: a checkpoint as ``cfg.tensor_shapes`` names it (None: random weights)."""
        super().__init__()
        if tensors is None:
            tensors = random_tensors(cfg, device=device)
        want = cfg.tensor_shapes()
        bad = [k for k, s in want.items() if k not in tensors or tuple(tensors[k].shape) != tuple(s)]
        if bad:
            raise ValueError(f"checkpoint tensors missing or of another shape: {bad[:5]}")
        self.cfg, self.dtype = cfg, dtype
        self.device = torch.device(device)
        self.embed = _frozen(tensors["embed"].to(device, dtype).contiguous())
        self.head = _frozen(tensors["head"].to(device, dtype).contiguous())
        around_one = lambda name: 1.0 + tensors[name].to(device).float()
        self.norm_f = _frozen(around_one("final.norm").contiguous())
        rotations: dict = {}
        self.layers = nn.ModuleList()
        for i, l in enumerate(cfg.layers):
            t = {k[len(f"l{i}.mix."):]: v for k, v in tensors.items() if k.startswith(f"l{i}.mix.")}
            if l.kind == "attention":
                mixer = BlockAttention(l.mixer, t, cfg.norm_eps, device, dtype, rotations)
            else:
                mixer = RECURRENT[l.kind](l.mixer, t, cfg.norm_eps, device, dtype)
            mlp = None
            if l.mlp is not None:
                mlp = GatedMLP({k: tensors[f"l{i}.mlp.{k}"] for k in ("gate", "up", "down")}, device, dtype, act="relu")
            self.layers.append(ParallelLayer(mixer, mlp, t["o"], around_one(f"l{i}.norm1"), around_one(f"l{i}.norm2") if mlp else None, device, dtype))

    # ------------------------------------------------------------ what an engine asks of a model
    def new_cache(self, batch: int, max_seq_len: int, page_size: int, n_pages: int | None = None) -> HybridCache:
        layers = []
        for l in self.cfg.layers:
            s = l.mixer
            if l.kind != "attention":
                layers.append(StateShape(s.heads, s.dim, s.vdim))
            else:
                layers.append(KvShape(s.kv_heads, s.dim, s.vdim) if s.kv_from is None else s.kv_from)
        return HybridCache(layers, batch, max_seq_len, page_size, self.device, self.dtype, n_pages)

    def vocab(self) -> int:
        return self.cfg.vocab_size

    def stream(self, batch, cache, keep=None) -> torch.Tensor:
        """The residual stream [N, width] (fp32) of the tokens of ``batch`` after the last layer; keys, values and states
        go to ``cache``.  keep: a list that receives a copy after every layer."""
        c, dt = self.cfg, self.dtype
        x = torch.empty(batch.ids.shape[0], c.width, dtype=torch.float32, device=self.device)
        weights = [(l.norm1, l.norm2) for l in self.layers] + [(None, None)]
        h1, h2 = S.stream_norms(x, c.norm_eps, dt, *weights[0], ids=batch.ids, table=self.embed)
        for i, l in enumerate(self.layers):
            y = l(h1, h2, batch, cache, i)
            h1, h2 = S.stream_norms(x, c.norm_eps, dt, *weights[i + 1], y=y, mult=c.residual_mult)
            if keep is not None:
                keep.append(x.clone())
        return x

    def logits(self, x: torch.Tensor, rows: torch.Tensor | None = None) -> torch.Tensor:
        """fp32 logits of the stream's rows (all, or those named)."""
        h = S.rms_rows(x, self.norm_f, self.cfg.norm_eps, self.dtype, rows)
        return S.softcap(linear(h, self.head, out_dtype=torch.float32), self.cfg.logit_softcap)

    def num_params(self) -> int:
        return sum(p.numel() for p in self.parameters())

    # ------------------------------------------------------------ folders
    @classmethod
    def from_folder(cls, path: str, device="cpu", dtype=torch.bfloat16) -> "Nufalorn":
        from ..io.safetensors import load_safetensors
        tensors = load_safetensors(os.path.join(path, "model.safetensors"))
        with open(os.path.join(path, "config.json")) as f:
            cfg = NufalornConfig.from_dict(json.load(f), {k: tuple(v.shape) for k, v in tensors.items()})
        return cls(cfg, tensors, device, dtype)
