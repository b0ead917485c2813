"""Ginisun: a decoder with latent attention, a mixture of clamped gated experts in every feed-forward, several residual streams
("hyper-connections") and Dynamic Tanh norms.

``config.json`` carries a list of layers, each with its own mixer and feed-forward sizes; tensors are named ``l<i>.mix.*``, ``l<i>.mlp.*``,
``l<i>.hc<q>.*`` (see :meth:`GinisunConfig.tensor_shapes`). The model runs inside :class:`~ferrotorch_b200.models.serving.ServingEngine`:

* prompts (any ragged batch): tcgen05 GEMMs, ragged flash attention on keys and values expanded from the latent, grouped expert GEMMs; everything
  between two projections is one pass over the f32 streams;
* decode (bf16, up to 16 sequences): split-K weight streaming, absorbed latent attention over the page cache, streamed experts -- ten launches a layer,
  replayed from one CUDA graph;
* f32: the same structure on exact FMA-pipe products and a plain attention kernel.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field
from pathlib import Path
from typing import Dict, List, Optional, Tuple

import torch

from .. import _lib
from ..errors import InvalidArgument
from ..ops.latent_attention import (LatentDecodeBuffers, LatentDims, LatentWeights, latent_attention_decode, latent_attention_rows, rotary_pair_tables)
from ..ops.moe import ExpertStack, MoeSmallBuffers, MoeWeights, linear_rows, moe_rows, moe_small
from ..ops.streams import DynamicTanhWeights, HyperWeights, SublayerOutput, hyper_embed, hyper_update, round_up
from .llama_infer import PAD_ROWS, _SplitKGemm
from .registry import checked_weights

EXPERT_SLOPE = 1.702          # g * sigmoid(1.702 g): fixed by the design
MAX_STREAMS = 16


@dataclass
class LatentMixerConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rope_base: float

    @staticmethod
    def from_dict(d: dict) -> "LatentMixerConfig":
        rot = d["rot"]
        if int(rot["dims"]) != int(d["rot_dim"]):
            raise InvalidArgument(f"Ginisun: rot.dims ({rot['dims']}) must equal rot_dim ({d['rot_dim']})")
        return LatentMixerConfig(int(d["heads"]), int(d["dim"]), int(d["rot_dim"]), int(d["vdim"]), int(d["kv_rank"]), float(d["scale"]), float(rot["base"]))

    def to_dict(self) -> dict:
        return dict(heads=self.heads, dim=self.dim, rot_dim=self.rot_dim, vdim=self.vdim, kv_rank=self.kv_rank, scale=self.scale,
                    rot=dict(base=self.rope_base, dims=self.rot_dim))


@dataclass
class ExpertConfig:
    ff: int
    limit: float = math.inf

    @staticmethod
    def from_dict(d: dict) -> "ExpertConfig":
        return ExpertConfig(int(d["ff"]), math.inf if d.get("limit") is None else float(d["limit"]))

    def to_dict(self) -> dict:
        return dict(ff=self.ff, limit=self.limit if math.isfinite(self.limit) else None)


@dataclass
class MoeConfig:
    """``groups`` (0: none), of which ``keep`` stay, and ``scale`` belong to routers that choose within the best groups of experts and norm their weights."""
    experts: int
    top: int
    expert: ExpertConfig
    shared: Optional[ExpertConfig] = None
    groups: int = 0
    keep: int = 0
    scale: float = 1.0

    @staticmethod
    def from_dict(d: dict) -> "MoeConfig":
        if d.get("kind", "moe") != "moe":
            raise InvalidArgument(f"unknown feed-forward kind {d['kind']!r}")
        r = d["router"]
        g = r.get("groups") or {}
        return MoeConfig(int(r["experts"]), int(r["top"]), ExpertConfig.from_dict(d["expert"]), ExpertConfig.from_dict(d["shared"]) if d.get("shared") else None,
                         int(g.get("count", 0)), int(g.get("keep", 0)), float(r.get("scale", 1.0)))

    def to_dict(self) -> dict:
        out = dict(kind="moe", router=dict(experts=self.experts, top=self.top), expert=self.expert.to_dict())
        if self.scale != 1.0:
            out["router"]["scale"] = self.scale
        if self.groups:
            out["router"]["groups"] = dict(count=self.groups, keep=self.keep)
        if self.shared:
            out["shared"] = self.shared.to_dict()
        return out


@dataclass
class GinisunLayer:
    mixer: LatentMixerConfig
    mlp: Optional[MoeConfig] = None

    @staticmethod
    def from_dict(d: dict) -> "GinisunLayer":
        if d["type"] != "latent_attention":
            raise InvalidArgument(f"Ginisun: unknown mixer {d['type']!r}")
        return GinisunLayer(LatentMixerConfig.from_dict(d["mixer"]), MoeConfig.from_dict(d["mlp"]) if d.get("mlp") else None)

    def to_dict(self) -> dict:
        return dict(type="latent_attention", mixer=self.mixer.to_dict(), mlp=self.mlp.to_dict() if self.mlp else None)


@dataclass
class GinisunConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    layers: List[GinisunLayer] = field(default_factory=list)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def from_dict(src) -> "GinisunConfig":
        """From a parsed ``config.json`` or its path."""
        d = src if isinstance(src, dict) else json.loads(Path(src).read_text())
        c = GinisunConfig(int(d["vocab"]), int(d["width"]), int(d.get("streams", 1)), float(d["norm"]["eps"]), [GinisunLayer.from_dict(x) for x in d["layers"]])
        c.validate()
        return c

    def to_dict(self) -> dict:
        return dict(architecture="Ginisun", vocab=self.vocab, width=self.width, streams=self.streams, norm=dict(eps=self.eps),
                    layers=[x.to_dict() for x in self.layers])

    def validate(self) -> None:
        if min(self.vocab, self.width, self.streams, len(self.layers)) < 1:
            raise InvalidArgument("Ginisun: vocab, width, streams and the number of layers must be positive")
        if self.streams > MAX_STREAMS:
            raise InvalidArgument(f"Ginisun: the stream kernels take up to {MAX_STREAMS} streams, got {self.streams}")
        for i, l in enumerate(self.layers):
            m = l.mixer
            if min(m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank) < 1 or m.rot_dim % 2:
                raise InvalidArgument(f"Ginisun: layer {i}: mixer sizes must be positive and rot_dim even")
            if not m.scale > 0:
                raise InvalidArgument(f"Ginisun: layer {i}: scale must be positive")
            if l.mlp and not 1 <= l.mlp.top <= l.mlp.experts:
                raise InvalidArgument(f"Ginisun: layer {i}: top must be between 1 and the number of experts")
            if l.mlp and (l.mlp.groups or l.mlp.scale != 1.0):
                raise InvalidArgument(f"Ginisun: layer {i}: the router has no groups and no scale")

    @staticmethod
    def uniform(layers: int, vocab: int, width: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, experts: int, top: int, ff: int, shared_ff: int = 0,
                streams: int = 4, limit: float = 7.0, rope_base: float = 10000.0, eps: float = 1e-5) -> "GinisunConfig":
        """``layers`` equal layers."""
        m = LatentMixerConfig(heads, dim, rot_dim, vdim, kv_rank, (dim + rot_dim) ** -0.5, rope_base)
        f = MoeConfig(experts, top, ExpertConfig(ff, limit), ExpertConfig(shared_ff, limit) if shared_ff else None) if experts else None
        c = GinisunConfig(vocab, width, streams, eps, [GinisunLayer(m, f) for _ in range(layers)])
        c.validate()
        return c

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        W, n = self.width, self.streams
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab, W), "head": (self.vocab, W)}

        def norm(name):
            out.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})
        norm("embed.norm")
        norm("final.norm")
        for i, l in enumerate(self.layers):
            p, m = f"l{i}.", l.mixer
            norm(p + "norm1")
            out.update({p + "mix.q": (m.heads * (m.dim + m.rot_dim), W), p + "mix.dkv": (m.kv_rank + m.rot_dim, W), p + "mix.dkv.norm": (m.kv_rank,),
                        p + "mix.uk": (m.heads * m.dim, m.kv_rank), p + "mix.uv": (m.heads * m.vdim, m.kv_rank), p + "mix.o": (W, m.heads * m.vdim)})
            subs = [1]
            if l.mlp:
                subs.append(2)
                norm(p + "norm2")
                out[p + "mlp.router"] = (l.mlp.experts, W)
                named = [(f"e{e}", l.mlp.expert.ff) for e in range(l.mlp.experts)] + ([("shared", l.mlp.shared.ff)] if l.mlp.shared else [])
                for nm, f in named:
                    out.update({f"{p}mlp.{nm}.gate": (f, W), f"{p}mlp.{nm}.up": (f, W), f"{p}mlp.{nm}.down": (W, f)})
            for q in subs:
                out.update({f"{p}hc{q}.in": (n,), f"{p}hc{q}.out": (n,), f"{p}hc{q}.mix": (n, n)})
        return out


class RandomGinisunWeights:
    """Random weights made tensor by tensor when they are asked for (large configurations never exist twice in memory)."""

    def __init__(self, cfg: GinisunConfig, device="cuda", seed: int = 0):
        self.cfg, self.device = cfg, device
        self.shapes = cfg.tensor_shapes()
        self.gen = torch.Generator(device=device).manual_seed(seed)

    def keys(self):
        return self.shapes.keys()

    def __contains__(self, k) -> bool:
        return k in self.shapes

    def __getitem__(self, name: str) -> torch.Tensor:
        s = self.shapes[name]
        t = torch.randn(s, device=self.device, generator=self.gen)
        if name.endswith(".alpha"):
            t = 0.5 + 0.05 * t
        elif name.endswith(".in"):
            t = 1.0 / s[0] + 0.05 * t
        elif name.endswith(".out"):
            t = 1.0 + 0.1 * t
        elif ".hc" in name:
            t = torch.eye(s[0], device=self.device) + 0.05 * t
        elif len(s) == 1:
            t = 0.05 * t + (0.0 if name.endswith(".b") else 1.0)
        elif name != "embed":
            t = t / math.sqrt(s[1])
        return t.to(torch.bfloat16)


@dataclass
class _Sub:
    """One sublayer: its connection weights, the norm ahead of it, and its weights (exactly one of ``attn`` and ``moe``)."""
    layer: int
    hyper: HyperWeights
    norm: DynamicTanhWeights
    attn: Optional[LatentWeights] = None
    moe: Optional[MoeWeights] = None
    g_proj: Optional[_SplitKGemm] = None
    g_out: Optional[_SplitKGemm] = None
    tables: Tuple[torch.Tensor, torch.Tensor] = None
    buffers: Optional[LatentDecodeBuffers] = None
    last_of_layer: bool = False


class GinisunModel:
    """Weights and layer schedule; ``weights`` maps the names of :meth:`GinisunConfig.tensor_shapes` to tensors (anything with ``[]`` and ``in``)."""

    def __init__(self, cfg: GinisunConfig, weights, device="cuda", dtype: torch.dtype = torch.bfloat16):
        cfg.validate()
        if dtype not in (torch.bfloat16, torch.float32):
            raise InvalidArgument("Ginisun runs in bfloat16 or float32")
        self.cfg, self.device, self.dtype, self.vocab = cfg, torch.device(device), dtype, cfg.vocab
        if self.device.type != "cuda":
            raise InvalidArgument("Ginisun runs on a CUDA device (its operators are CUDA kernels)")
        self._load(weights)

    # -- weights ---------------------------------------------------------------
    def _load(self, weights) -> None:
        cfg, dev, dt = self.cfg, self.device, self.dtype
        get = checked_weights("Ginisun", cfg.tensor_shapes(), weights, dev)

        def norm(name):
            return DynamicTanhWeights.from_tensors(get(name + ".alpha"), get(name), get(name + ".b"), dev)

        def matrix(t, ld):
            m = torch.zeros(t.shape[0], round_up(t.shape[1], ld), device=dev, dtype=dt)
            m[:, : t.shape[1]] = t
            return m[:, : t.shape[1]]
        W = cfg.width
        self.embed, self.head = matrix(get("embed"), 8), matrix(get("head"), 8)
        self.embed_norm, self.final_norm = norm("embed.norm"), norm("final.norm")
        self.subs: List[_Sub] = []
        for i, l in enumerate(cfg.layers):
            p, m = f"l{i}.", l.mixer

            def hyper(q):
                return HyperWeights.from_tensors(get(f"{p}hc{q}.in"), get(f"{p}hc{q}.mix"), get(f"{p}hc{q}.out"), dev)
            dims = LatentDims(m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, cfg.eps)
            aw = LatentWeights.pack(dims, *(get(p + "mix." + k) for k in ("q", "dkv", "dkv.norm", "uk", "uv", "o")), dev, dt)
            self.subs.append(_Sub(i, hyper(1), norm(p + "norm1"), attn=aw))
            if l.mlp:
                f = l.mlp

                def stack(names, e):
                    cols = [[get(f"{p}mlp.{nm}.{k}") for nm in names] for k in ("gate", "up", "down")]
                    return ExpertStack.pack(*cols, e.limit, dev, dt)
                mw = MoeWeights(matrix(get(p + "mlp.router"), 8), stack([f"e{e}" for e in range(f.experts)], f.expert),
                                stack(["shared"], f.shared) if f.shared else None, W, f.top, EXPERT_SLOPE)
                self.subs.append(_Sub(i, hyper(2), norm(p + "norm2"), moe=mw))
            self.subs[-1].last_of_layer = True
        self._ld = round_up(W, 8)

    @property
    def cache_rows(self) -> List[int]:
        return [s.attn.dims.row for s in self.subs if s.attn]

    def prepare(self, max_positions: int) -> None:
        """Rotation tables for positions below ``max_positions``."""
        made: dict = {}
        for s in self.subs:
            if s.attn:
                m = self.cfg.layers[s.layer].mixer
                key = (m.rot_dim, m.rope_base)
                if key not in made:
                    made[key] = rotary_pair_tables(max_positions, m.rot_dim, m.rope_base, self.device)
                s.tables = made[key]

    # -- prompts and any ragged batch ------------------------------------------
    @torch.no_grad()
    def forward_rows(self, batch, cache, taps: Optional[list] = None) -> Optional[torch.Tensor]:
        """Runs the new tokens of a :class:`RowBatch`, writes their cache rows and returns the logits of ``batch.want`` (``None`` if empty). ``taps``
        collects the sum of the streams after every layer, ``[rows, width]``."""
        cfg, T, W = self.cfg, batch.rows, self.cfg.width
        x = torch.empty(T, cfg.streams, self._ld, device=self.device, dtype=torch.float32)
        h = torch.empty(T, self._ld, device=self.device, dtype=self.dtype)[:, :W]
        first = self.subs[0]
        hyper_embed(batch.ids, self.embed, self.embed_norm, x, first.hyper.inp, first.norm, h, T, W)
        for k, s in enumerate(self.subs):
            if s.attn:
                y = latent_attention_rows(h, s.attn, batch, cache.rows[s.layer], *s.tables)
            else:
                y = moe_rows(h, s.moe)
            last = k + 1 == len(self.subs)
            nxt = None if last else self.subs[k + 1]
            hyper_update(x, s.hyper, y, None if last else nxt.hyper.inp, self.final_norm if last else nxt.norm, h, T, W, store=not last or taps is not None)
            if taps is not None and s.last_of_layer:
                taps.append(x.sum(1)[:, :W].clone())
        if batch.want is None:
            return None
        hw = torch.empty(batch.want.numel(), self._ld, device=self.device, dtype=self.dtype)[:, :W]
        hw.copy_(h[batch.want])
        return linear_rows(hw, self.head, out_f32=True)

    # -- decode ------------------------------------------------------------------
    def decode_supported(self) -> bool:
        """Whether the captured decode step covers this model: bf16, and sizes within the streaming kernels' shared memory."""
        return self.dtype == torch.bfloat16 and all(s.attn.dims.decode_supported() if s.attn else s.moe.small_supported() for s in self.subs)

    def decode_begin(self, max_batch: int, max_tokens: int) -> None:
        """Allocates the decode step's buffers."""
        cfg, dev, W = self.cfg, self.device, self.cfg.width
        planes: dict = {}
        shared: Dict[LatentDims, LatentDecodeBuffers] = {}
        for s in self.subs:
            if s.attn:
                if s.attn.dims not in shared:
                    shared[s.attn.dims] = LatentDecodeBuffers(s.attn.dims, max_batch, max_tokens, dev)
                s.buffers = shared[s.attn.dims]
                s.g_proj, s.g_out = _SplitKGemm(s.attn.proj, dev, planes), _SplitKGemm(s.attn.out, dev, planes)
        self._g_head = _SplitKGemm(self.head, dev)
        moes = [s.moe for s in self.subs if s.moe]
        self._moe_buffers = MoeSmallBuffers.allocate(moes, dev) if moes else None
        self._x = torch.zeros(PAD_ROWS, cfg.streams, self._ld, device=dev)
        self._h = torch.zeros(PAD_ROWS, self._ld, device=dev, dtype=self.dtype)[:, :W]
        self._logits = torch.zeros(PAD_ROWS, round_up(self.vocab, 4), device=dev)[:, : self.vocab]

    @torch.no_grad()
    def decode(self, state, B: int, cache) -> torch.Tensor:
        """One token for the first ``B`` sequences of ``state``; returns the logits buffer ``[16, vocab]`` (rows below ``B`` are valid)."""
        W, x, h = self.cfg.width, self._x, self._h
        first = self.subs[0]
        hyper_embed(state.tokens, self.embed, self.embed_norm, x, first.hyper.inp, first.norm, h, B, W)
        for k, s in enumerate(self.subs):
            if s.attn:
                s.g_proj(h)
                g = s.g_proj
                a = latent_attention_decode(g.planes, g.splits, s.attn, s.buffers, state, cache.rows[s.layer], *s.tables, B)
                s.g_out(a)
                y = SublayerOutput(planes=s.g_out.planes)
            else:
                y = moe_small(h, s.moe, self._moe_buffers, B)
            last = k + 1 == len(self.subs)
            nxt = None if last else self.subs[k + 1]
            hyper_update(x, s.hyper, y, None if last else nxt.hyper.inp, self.final_norm if last else nxt.norm, h, B, W, store=not last)
        self._g_head(h)
        g = self._g_head
        _lib.call("ft_splitk_reduce", g.planes, g.splits, B, self.vocab, g.ldp, g.plane_stride, None, self._logits, self._logits.stride(0), 1, _lib.S())
        return self._logits
