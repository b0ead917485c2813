"""Mepupel: a decoder whose layers have one of three mixers (a Mamba-2 state space, grouped-query attention with a window and kept first tokens, latent attention without
positions, whose latent later layers may share) beside a dense or mixture-of-experts feed-forward that reads the same residual through a norm of its own.

``config.json`` carries a list of layers, each with its own mixer and feed-forward sizes; tensors are named ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.norm1`` and ``l<i>.norm2`` (see
:meth:`MepupelConfig.tensor_shapes`). The model runs inside :class:`~ferrotorch_b200.models.serving.ServingEngine`:

* prompts (any ragged batch): one tcgen05 GEMM for all projections of a mixer (a second, small one with f32 results for the step sizes of a state space), ragged flash attention
  over the pages or on keys and values expanded from the latent, the chunked walk of the state space, grouped expert GEMMs; one pass over the residual per layer, which
  leaves the operands of the next mixer and the next feed-forward;
* decode (bf16, up to 16 sequences): split-K weight streaming, whose partial sums every kernel behind it consumes directly, streamed experts -- replayed from one CUDA graph;
* f32: the same structure on exact FMA-pipe products, plain attention kernels and the state space token by token.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field
from pathlib import Path
from typing import Dict, List, Optional, Tuple, Union

import torch

from .. import _lib
from ..errors import InvalidArgument
from ..ops.gqa_attention import GqaDecodeBuffers, GqaDims, GqaWeights, gqa_attention_decode, gqa_attention_rows, pack_head_columns, pack_head_rows
from ..ops.latent_attention import (LatentDecodeBuffers, LatentDims, LatentWeights, latent_attention_decode, latent_attention_rows, latent_context, rotary_pair_tables)
from ..ops.moe import ExpertStack, MoeSmallBuffers, MoeWeights, RouteRule, linear_rows, moe_rows, moe_small
from ..ops.residual import DenseGatedWeights, dense_gated_rows, gated_act_planes, parallel_embed, parallel_update
from ..ops.state_space import SsmDecodeBuffers, SsmDims, SsmWeights, state_space_decode, state_space_rows
from ..ops.streams import SublayerOutput, padded_vector, round_up
from .ginisun import ExpertConfig, MoeConfig
from .llama_infer import PAD_ROWS, _SplitKGemm
from .pufevik import AttentionConfig
from .registry import checked_weights

ACTIVATION = "silu"                  # fixed by the design


@dataclass
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int

    @staticmethod
    def from_dict(d: dict) -> "Mamba2Config":
        return Mamba2Config(*(int(d[k]) for k in ("heads", "vdim", "state", "groups", "norm_groups", "conv")))

    def to_dict(self) -> dict:
        return dict(heads=self.heads, vdim=self.vdim, state=self.state, groups=self.groups, norm_groups=self.norm_groups, conv=self.conv)

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    def dims(self, eps: float) -> SsmDims:
        return SsmDims(self.heads, self.vdim, self.state, self.groups, self.conv, self.norm_groups, eps)

    def validate(self, where: str) -> None:
        try:
            self.dims(1.0).validate()
        except InvalidArgument as e:
            raise InvalidArgument(f"{where}: {e}") from None


@dataclass
class LatentConfig:
    """Latent attention without positions; ``kv_from``: the earlier layer whose latent this one reads."""
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    kv_from: Optional[int] = None

    @staticmethod
    def from_dict(d: dict) -> "LatentConfig":
        return LatentConfig(int(d["heads"]), int(d["dim"]), int(d["vdim"]), int(d["q_rank"]), int(d["kv_rank"]), float(d["scale"]),
                            None if d.get("kv_from") is None else int(d["kv_from"]))

    def to_dict(self) -> dict:
        d = dict(heads=self.heads, dim=self.dim, vdim=self.vdim, q_rank=self.q_rank, kv_rank=self.kv_rank, scale=self.scale)
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d

    def dims(self, eps: float) -> LatentDims:
        return LatentDims(self.heads, self.dim, 0, self.vdim, self.kv_rank, self.scale, eps, self.q_rank, self.kv_from is None)

    def validate(self, where: str) -> None:
        if min(self.heads, self.dim, self.vdim, self.q_rank, self.kv_rank) < 1 or not self.scale > 0:
            raise InvalidArgument(f"{where}: sizes and scale must be positive")


@dataclass
class DenseConfig:
    ff: int

    def to_dict(self) -> dict:
        return dict(kind="dense", ff=self.ff)


Mixer = Union[Mamba2Config, AttentionConfig, LatentConfig]
MIXERS = {"mamba2": Mamba2Config, "attention": AttentionConfig, "latent_attention": LatentConfig}


@dataclass
class MepupelLayer:
    mixer: Mixer
    mlp: Union[DenseConfig, MoeConfig, None] = None

    @staticmethod
    def from_dict(d: dict) -> "MepupelLayer":
        if d["type"] not in MIXERS:
            raise InvalidArgument(f"Mepupel: unknown mixer {d['type']!r}")
        f = d.get("mlp")
        if f and f.get("kind") == "dense":
            mlp = DenseConfig(int(f["ff"]))
        else:
            mlp = MoeConfig.from_dict(f) if f else None
        return MepupelLayer(MIXERS[d["type"]].from_dict(d["mixer"]), mlp)

    @property
    def type(self) -> str:
        return next(k for k, c in MIXERS.items() if isinstance(self.mixer, c))

    def to_dict(self) -> dict:
        return dict(type=self.type, mixer=self.mixer.to_dict(), mlp=self.mlp.to_dict() if self.mlp else None)


@dataclass
class MepupelConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    layers: List[MepupelLayer] = field(default_factory=list)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def from_dict(src) -> "MepupelConfig":
        """From a parsed ``config.json`` or its path."""
        d = src if isinstance(src, dict) else json.loads(Path(src).read_text())
        c = MepupelConfig(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["residual_mult"]), [MepupelLayer.from_dict(x) for x in d["layers"]])
        c.validate()
        return c

    def to_dict(self) -> dict:
        return dict(architecture="Mepupel", vocab=self.vocab, width=self.width, norm=dict(eps=self.eps), residual_mult=self.residual_mult, layers=[x.to_dict() for x in self.layers])

    def latent_source(self, i: int) -> int:
        """The layer whose cached latent layer ``i`` reads."""
        f = self.layers[i].mixer.kv_from
        return i if f is None else f

    def validate(self) -> None:
        if min(self.vocab, self.width, len(self.layers)) < 1:
            raise InvalidArgument("Mepupel: vocab, width and the number of layers must be positive")
        for i, l in enumerate(self.layers):
            where, m, f = f"Mepupel: layer {i}", l.mixer, l.mlp
            m.validate(where)
            if isinstance(m, AttentionConfig) and m.v_mix:
                raise InvalidArgument(f"{where}: values are not mixed")
            if isinstance(m, LatentConfig) and m.kv_from is not None:
                j = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if not isinstance(j, LatentConfig) or j.kv_from is not None or j.kv_rank != m.kv_rank:
                    raise InvalidArgument(f"{where}: kv_from must name an earlier latent_attention layer with a latent of its own and the same kv_rank")
            if isinstance(f, DenseConfig) and f.ff < 1:
                raise InvalidArgument(f"{where}: mlp.ff must be positive")
            if isinstance(f, MoeConfig):
                if not 1 <= f.top <= f.experts or min(f.expert.ff, f.shared.ff if f.shared else 1) < 1:
                    raise InvalidArgument(f"{where}: router.top must be between 1 and router.experts, the experts' sizes positive")
                if f.groups and (f.groups < 1 or f.experts % f.groups or not 1 <= f.keep <= f.groups or f.top > f.keep * (f.experts // f.groups)):
                    raise InvalidArgument(f"{where}: router.groups must split the experts evenly and keep enough of them for router.top")
                if any(math.isfinite(e.limit) for e in (f.expert, f.shared) if e):
                    raise InvalidArgument(f"{where}: experts have no limit")

    @staticmethod
    def pattern(kinds: str, vocab: int, width: int, ssm: dict, attention: dict, latent: dict, mlp: Union[DenseConfig, MoeConfig, None], first_ff: int = 0,
                residual_mult: float = 1.0, eps: float = 1e-5) -> "MepupelConfig":
        """Layers by letter: ``m`` (state space), ``a`` (attention), ``l`` (latent attention), ``s`` (latent attention on the latent of the ``l`` before it), each kind with the
        sizes of its dictionary (as in ``config.json``) and all with the same feed-forward, but for a dense one of ``first_ff`` neurons in the first layer."""
        layers = []
        for i, k in enumerate(kinds):
            f = DenseConfig(first_ff) if first_ff and i == 0 else mlp
            if k in "ls":
                layers.append(MepupelLayer(LatentConfig(**latent, kv_from=kinds.rindex("l", 0, i) if k == "s" else None), f))
            else:
                layers.append(MepupelLayer(Mamba2Config(**ssm) if k == "m" else AttentionConfig.from_dict(attention), f))
        c = MepupelConfig(vocab, width, eps, residual_mult, layers)
        c.validate()
        return c

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        W = self.width
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab, W), "head": (self.vocab, W), "final.norm": (W,)}
        for i, l in enumerate(self.layers):
            p, m, f = f"l{i}.", l.mixer, l.mlp
            q = p + "mix."
            out[p + "norm1"] = (W,)
            if isinstance(m, Mamba2Config):
                out.update({q + "in": (m.inner + m.channels + m.heads, W), q + "conv": (m.channels, m.conv), q + "conv.b": (m.channels,), q + "dt_bias": (m.heads,),
                            q + "A_log": (m.heads,), q + "D": (m.heads,), q + "norm": (m.inner,), q + "o": (W, m.inner)})
            elif isinstance(m, AttentionConfig):
                out.update({q + "q": (m.heads * m.dim, W), q + "k": (m.kv_heads * m.dim, W), q + "v": (m.kv_heads * m.vdim, W), q + "o": (W, m.heads * m.vdim)})
            else:
                out.update({q + "dq": (m.q_rank, W), q + "dq.norm": (m.q_rank,), q + "uq": (m.heads * m.dim, m.q_rank), q + "uk": (m.heads * m.dim, m.kv_rank),
                            q + "uv": (m.heads * m.vdim, m.kv_rank), q + "o": (W, m.heads * m.vdim)})
                if m.kv_from is None:
                    out.update({q + "dkv": (m.kv_rank, W), q + "dkv.norm": (m.kv_rank,)})
            q = p + "mlp."
            if f:
                out[p + "norm2"] = (W,)
            if isinstance(f, DenseConfig):
                out.update({q + "gate": (f.ff, W), q + "up": (f.ff, W), q + "down": (W, f.ff), q + "gate.b": (f.ff,), q + "up.b": (f.ff,), q + "down.b": (W,)})
            elif f:
                out.update({q + "router": (f.experts, W), q + "correction": (f.experts,)})
                for nm, n in [(f"e{e}", f.expert.ff) for e in range(f.experts)] + ([("shared", f.shared.ff)] if f.shared else []):
                    out.update({f"{q}{nm}.gate": (n, W), f"{q}{nm}.up": (n, W), f"{q}{nm}.down": (W, n)})
        return out


class RandomMepupelWeights:
    """Random weights made tensor by tensor when they are asked for (large configurations never exist twice in memory)."""

    def __init__(self, cfg: MepupelConfig, device="cuda", seed: int = 0):
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
        if name.endswith(("norm", "norm1", "norm2", ".D")):
            t = 1.0 + 0.05 * t
        elif name.endswith(".dt_bias"):
            t = -3.0 + t
        elif len(s) == 2 and name != "embed":
            t = t / math.sqrt(s[1])
        elif name != "embed" and not name.endswith(".A_log"):
            t = 0.05 * t
        return t.to(torch.bfloat16)


@dataclass
class _Layer:
    """Weights of one layer. Of ``attn``, ``latent`` and ``ssm`` one is set, of ``dense`` and ``moe`` at most one. ``proj`` and ``out`` are the mixer's first and last product."""
    norm1: torch.Tensor
    proj: torch.Tensor
    out: torch.Tensor
    attn: Optional[GqaWeights] = None
    latent: Optional[LatentWeights] = None
    ssm: Optional[SsmWeights] = None
    source: int = 0                      # the layer whose cache rows the mixer reads
    lends: bool = False                  # later layers read this one's latent
    norm2: Optional[torch.Tensor] = None
    dense: Optional[DenseGatedWeights] = None
    moe: Optional[MoeWeights] = None
    tables: Tuple[Optional[torch.Tensor], Optional[torch.Tensor]] = (None, None)
    buffers: object = None
    mixed: Optional[torch.Tensor] = None
    g_proj: Optional[_SplitKGemm] = None
    g_out: Optional[_SplitKGemm] = None
    g_expand: Optional[_SplitKGemm] = None
    g_gu: Optional[_SplitKGemm] = None
    g_down: Optional[_SplitKGemm] = None

    @property
    def mixer(self):
        return self.attn or self.latent or self.ssm


class MepupelModel:
    """Weights and layer schedule; ``weights`` maps the names of :meth:`MepupelConfig.tensor_shapes` to tensors (anything with ``[]``, ``in`` and ``keys``)."""

    def __init__(self, cfg: MepupelConfig, weights, device="cuda", dtype: torch.dtype = torch.bfloat16):
        cfg.validate()
        if dtype not in (torch.bfloat16, torch.float32):
            raise InvalidArgument("Mepupel runs in bfloat16 or float32")
        self.cfg, self.device, self.dtype, self.vocab = cfg, torch.device(device), dtype, cfg.vocab
        self.side_by_side = True             # decode: the two sublayers of a layer on two streams
        if self.device.type != "cuda":
            raise InvalidArgument("Mepupel runs on a CUDA device (its operators are CUDA kernels)")
        self._load(weights)

    # -- weights ---------------------------------------------------------------
    def _load(self, weights) -> None:
        cfg, dev, dt, W = self.cfg, self.device, self.dtype, self.cfg.width
        get = checked_weights("Mepupel", cfg.tensor_shapes(), weights, dev)

        def matrix(t):
            m = torch.zeros(t.shape[0], round_up(t.shape[1], 32), device=dev, dtype=dt)
            m[:, : t.shape[1]] = t
            return m[:, : t.shape[1]]

        def vector(name):
            return padded_vector(get(name), dev)
        self.embed, self.head, self.final_norm = matrix(get("embed")), matrix(get("head")), vector("final.norm")
        lenders = {l.mixer.kv_from for l in cfg.layers if isinstance(l.mixer, LatentConfig)}
        self.layers: List[_Layer] = []
        for i, l in enumerate(cfg.layers):
            p, m, f = f"l{i}.", l.mixer, l.mlp
            q, norm1 = p + "mix.", vector(p + "norm1")
            if isinstance(m, Mamba2Config):
                D = m.dims(cfg.eps)
                w = SsmWeights.pack(D, *(get(q + k) for k in ("conv", "conv.b", "dt_bias", "A_log", "D", "norm")), dev)
                layer = _Layer(norm1, matrix(SsmWeights.pack_projection(D, get(q + "in"), dev, dt)), matrix(SsmWeights.pack_output(D, get(q + "o"), dev, dt)), ssm=w)
            elif isinstance(m, AttentionConfig):
                D = GqaDims(m.heads, m.kv_heads, m.dim, m.vdim, m.rot_dims, m.scale, cfg.eps, window=m.window, keep=m.keep_first if m.window else 0, halves=True, norm=False)
                rows = [pack_head_rows(get(q + k), n, s, dev, dt) for k, n, s in (("q", m.heads, m.dim), ("k", m.kv_heads, m.dim), ("v", m.kv_heads, m.vdim))]
                layer = _Layer(norm1, matrix(torch.cat(rows)), matrix(pack_head_columns(get(q + "o"), m.heads, m.vdim, dev, dt)), attn=GqaWeights.pack(D, None, None, dev))
            else:
                own = m.kv_from is None
                w = LatentWeights.pack(m.dims(cfg.eps), get(q + "uq"), get(q + "dkv") if own else None, get(q + "dkv.norm") if own else None, get(q + "uk"), get(q + "uv"), get(q + "o"),
                                       dev, dt, dq=get(q + "dq"), q_norm=get(q + "dq.norm"))
                layer = _Layer(norm1, w.proj, w.out, latent=w, source=cfg.latent_source(i), lends=i in lenders)
            if layer.latent is None:
                layer.source = i
            q = p + "mlp."
            if f:
                layer.norm2 = vector(p + "norm2")
            if isinstance(f, DenseConfig):
                layer.dense = DenseGatedWeights.pack(*(get(q + k) for k in ("gate", "up", "down")), dev, dt, ACTIVATION, *(get(f"{q}{k}.b") for k in ("gate", "up", "down")))
            elif f:
                def stack(names, e):
                    return ExpertStack.pack(*([get(f"{q}{nm}.{k}") for nm in names] for k in ("gate", "up", "down")), e.limit, dev, dt)
                rule = RouteRule(vector(q + "correction"), f.groups, f.keep, f.scale)
                layer.moe = MoeWeights(matrix(get(q + "router")), stack([f"e{e}" for e in range(f.experts)], f.expert), stack(["shared"], f.shared) if f.shared else None, W, f.top,
                                       form=ACTIVATION, rule=rule)
            self.layers.append(layer)
        self._ld = round_up(W, 8)

    @property
    def cache_rows(self) -> List[int]:
        return [l.attn.dims.row if l.attn else l.latent.dims.row if l.latent and l.latent.dims.own else 0 for l in self.layers]

    @property
    def state_sizes(self) -> List[int]:
        return [l.ssm.dims.state_size if l.ssm else 0 for l in self.layers]

    def prepare(self, max_positions: int) -> None:
        """Rotation tables for positions below ``max_positions``."""
        made: dict = {}
        for l, c in zip(self.layers, self.cfg.layers):
            if l.attn:
                a = c.mixer
                key = (a.rot_dims, a.rope_base, tuple(sorted(a.scaling.items())) if a.scaling else None)
                if key not in made:
                    made[key] = rotary_pair_tables(max_positions, a.rot_dims, a.rope_base, self.device, a.rope_scaling)
                l.tables = made[key]

    def _next_norms(self, k: int) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
        """Norm weights of layer ``k``'s operands; past the last layer the model's norm."""
        return (self.layers[k].norm1, self.layers[k].norm2) if k < len(self.layers) else (self.final_norm, None)

    # -- prompts and any ragged batch ------------------------------------------
    def _mix_rows(self, h: torch.Tensor, l: _Layer, batch, cache, i: int, contexts: dict) -> SublayerOutput:
        if l.latent:
            if l.lends and self.dtype == torch.bfloat16:
                contexts[i] = latent_context(l.latent.dims, batch, h.device, h.dtype)
            return latent_attention_rows(h, l.latent, batch, cache.rows[l.source], *l.tables, contexts.get(l.source))
        if l.ssm:
            D = l.ssm.dims
            a = state_space_rows(linear_rows(h, l.proj[: D.main]), linear_rows(h, l.proj[D.main:], out_f32=True), l.ssm, batch, cache.states.data[i])
        else:
            a = torch.empty(h.shape[0], l.out.shape[1], device=h.device, dtype=h.dtype)
            gqa_attention_rows(linear_rows(h, l.proj), l.attn, batch, cache.rows[i], *l.tables, None, a)
        y = linear_rows(a, l.out, out_f32=True)
        return SublayerOutput(planes=y.as_strided((1, y.shape[0], y.shape[1]), (0, y.stride(0), 1)))

    @torch.no_grad()
    def forward_rows(self, batch, cache, taps: Optional[list] = None) -> Optional[torch.Tensor]:
        """Runs the new tokens of a :class:`RowBatch`, writes their cache rows, advances the states and returns the logits of ``batch.want`` (``None`` if empty). ``taps``
        collects the residual after every layer, ``[rows, width]``."""
        cfg, T, W = self.cfg, batch.rows, self.cfg.width
        x = torch.empty(T, self._ld, device=self.device, dtype=torch.float32)
        h1, h2 = torch.empty(2, T, self._ld, device=self.device, dtype=self.dtype)[:, :, :W]
        parallel_embed(batch.ids, self.embed, *self._next_norms(0), cfg.eps, x, h1, h2, T)
        contexts: dict = {}
        for i, l in enumerate(self.layers):
            a = self._mix_rows(h1, l, batch, cache, i, contexts)
            b = dense_gated_rows(h2, l.dense) if l.dense else moe_rows(h2, l.moe) if l.moe else None
            last = i + 1 == len(self.layers)
            parallel_update(x, cfg.residual_mult, a, b, *self._next_norms(i + 1), cfg.eps, h1, h2, T, W, store=not last or taps is not None)
            if taps is not None:
                taps.append(x[:, :W].clone())
        if batch.want is None:
            return None
        hw = torch.empty(batch.want.numel(), self._ld, device=self.device, dtype=self.dtype)[:, :W]
        hw.copy_(h1[batch.want])
        return linear_rows(hw, self.head, out_f32=True)

    # -- decode ------------------------------------------------------------------
    def decode_supported(self) -> bool:
        """Whether the captured decode step covers this model: bf16, and sizes within its kernels' shared memory."""
        return self.dtype == torch.bfloat16 and all(l.mixer.dims.decode_supported() and (l.moe is None or l.moe.small_supported()) for l in self.layers)

    def decode_begin(self, max_batch: int, max_tokens: int) -> None:
        """Allocates the decode step's buffers."""
        dev, W = self.device, self.cfg.width
        planes: dict = {}
        shared: dict = {}
        rows: dict = {}

        def row_buffer(n):
            if n not in rows:
                rows[n] = torch.zeros(PAD_ROWS, n, device=dev, dtype=self.dtype)
            return rows[n]
        for l in self.layers:
            D = l.mixer.dims
            if D not in shared:
                shared[D] = SsmDecodeBuffers(D, dev) if l.ssm else (GqaDecodeBuffers if l.attn else LatentDecodeBuffers)(D, max_batch, max_tokens, dev)
            l.buffers = shared[D]
            if l.attn:
                l.mixed = row_buffer(D.out_cols)
            # the two sublayers of a layer hand their planes to the residual update together: each kind has planes of its own
            l.g_proj, l.g_out = _SplitKGemm(l.proj, dev, planes.setdefault("in", {})), _SplitKGemm(l.out, dev, planes.setdefault("mixer", {}))
            if l.latent:
                l.g_expand = _SplitKGemm(l.latent.uq, dev, planes.setdefault("expand", {}))
            if l.dense:
                l.g_gu, l.g_down = _SplitKGemm(l.dense.gu, dev, planes.setdefault("gate", {})), _SplitKGemm(l.dense.down, dev, planes.setdefault("feed-forward", {}))
        self._side = torch.cuda.Stream(dev)
        self._g_head = _SplitKGemm(self.head, dev)
        moes = [l.moe for l in self.layers if l.moe]
        self._moe_buffers = MoeSmallBuffers.allocate(moes, dev) if moes else None
        self._act = {n: torch.zeros(PAD_ROWS, n, device=dev, dtype=self.dtype) for n in {l.dense.fp for l in self.layers if l.dense}}
        self._x = torch.zeros(PAD_ROWS, self._ld, device=dev)
        self._h1, self._h2 = torch.zeros(2, PAD_ROWS, self._ld, device=dev, dtype=self.dtype)[:, :, :W]
        self._logits = torch.zeros(PAD_ROWS, round_up(self.vocab, 4), device=dev)[:, : self.vocab]

    def _mix_decode(self, l: _Layer, i: int, state, B: int, cache) -> SublayerOutput:
        g = l.g_proj
        g(self._h1)
        if l.ssm:
            a = state_space_decode(g.planes, g.splits, l.ssm, l.buffers, state, cache.states.data[i], B)
        elif l.attn:
            a = l.mixed
            gqa_attention_decode(g.planes, g.splits, l.attn, l.buffers, state, cache.rows[i], *l.tables, B, 0, a)
        else:
            a = latent_attention_decode(g.planes, g.splits, l.latent, l.buffers, state, cache.rows[l.source], *l.tables, B, l.g_expand)
        l.g_out(a)
        return SublayerOutput(planes=l.g_out.planes)

    def _feed_decode(self, l: _Layer, B: int) -> Optional[SublayerOutput]:
        if l.moe:
            return moe_small(self._h2, l.moe, self._moe_buffers, B)
        if not l.dense:
            return None
        d, a = l.dense, self._act[l.dense.fp]
        l.g_gu(self._h2)
        gated_act_planes(l.g_gu.planes, l.g_gu.splits, B, d.fp, d.act, a, d.gu_bias)
        l.g_down(a[:, : d.down.shape[1]])
        return SublayerOutput(planes=l.g_down.planes, bias=d.down_bias)

    @torch.no_grad()
    def decode(self, state, B: int, cache) -> torch.Tensor:
        """One token for the first ``B`` sequences of ``state``; returns the logits buffer ``[16, vocab]`` (rows below ``B`` are valid)."""
        cfg, W, x, h1, h2 = self.cfg, self.cfg.width, self._x, self._h1, self._h2
        parallel_embed(state.tokens, self.embed, *self._next_norms(0), cfg.eps, x, h1, h2, B)
        main, side, lib = torch.cuda.current_stream(self.device), self._side, _lib.kernels()
        for i, l in enumerate(self.layers):
            # the two sublayers of a layer do not depend on one another: the feed-forward streams its weights beside the mixer's chain of small kernels
            two = self.side_by_side and l.norm2 is not None
            if two:
                side.wait_stream(main)
                with torch.cuda.stream(side):
                    lib.ft_pdl_break()
                    b = self._feed_decode(l, B)
            a = self._mix_decode(l, i, state, B, cache)
            if two:
                main.wait_stream(side)
                lib.ft_pdl_break()
            else:
                b = self._feed_decode(l, B)
            parallel_update(x, cfg.residual_mult, a, b, *self._next_norms(i + 1), cfg.eps, h1, h2, B, W, store=i + 1 < len(self.layers))
        self._g_head(h1)
        g = self._g_head
        _lib.call("ft_splitk_reduce", g.planes, g.splits, B, self.vocab, g.ldp, g.plane_stride, None, self._logits, self._logits.stride(0), 1, _lib.S())
        return self._logits
