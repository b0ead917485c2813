"""Vemepel: a decoder whose layers have one of three mixers (differential attention within chunks, whose keys and values later layers may share; latent attention without
positions, gated per head; latent attention with a rotated part, gated per element) and a dense or mixture-of-experts feed-forward, with norms ahead of and behind every sublayer.
Ahead of a mixer every column is shifted towards the previous token, and what a layer hands on is a weighted sum of the results of all layers so far.

``config.json`` carries a list of layers, each with its own mixer and feed-forward sizes; tensors are named ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.norm1``, ``.norm1b``,
``.norm2``, ``.norm2b``, ``.shift`` and ``.dwa`` (see :meth:`VemepelConfig.tensor_shapes`). The model runs inside :class:`~ferrotorch_b200.models.serving.ServingEngine`:

* prompts (any ragged batch): one tcgen05 GEMM for all projections of a mixer, ragged flash attention over the pages (both maps of a differential head in one CTA) or on keys and
  values expanded from the latent, grouped expert GEMMs; one pass over the residual per sublayer, the one behind a layer reads the results of all layers along;
* decode (bf16, up to 16 sequences): split-K weight streaming, whose partial sums every kernel behind it consumes directly, streamed experts -- replayed from one CUDA graph;
* f32: the same structure on exact FMA-pipe products and plain attention kernels.

The previous token's operand is recurrent state: one f32 row per sequence and layer.
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
from ..ops.gqa_attention import (GATE_ELEMENT, GATE_HEAD, GqaDecodeBuffers, GqaDims, GqaWeights, differential_blend, gqa_attention_decode, gqa_attention_rows, pack_head_columns,
                                 pack_head_rows)
from ..ops.latent_attention import LatentDecodeBuffers, LatentDims, LatentWeights, latent_attention_decode, latent_attention_rows, rotary_pair_tables
from ..ops.moe import MAX_TOP, ExpertStack, MoeSmallBuffers, MoeWeights, RouteRule, linear_rows, moe_rows, moe_small
from ..ops.residual import DensePolyWeights, TokenShift, dense_poly_rows, depth_embed, depth_update, poly_norm_planes, residual_update, token_shift
from ..ops.streams import SublayerOutput, padded_vector, round_up
from .ginisun import MoeConfig
from .llama_infer import PAD_ROWS, _SplitKGemm
from .mepupel import DenseConfig
from .registry import checked_weights

ACTIVATION = "silu"                  # of the experts; fixed by the design


@dataclass
class DifferentialConfig:
    """Differential grouped-query attention within chunks of ``chunk`` positions (0: one chunk); ``kv_from``: the earlier layer whose keys and values this one reads."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    chunk: int = 0
    kv_from: Optional[int] = None

    @staticmethod
    def from_dict(d: dict) -> "DifferentialConfig":
        return DifferentialConfig(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]), float(d["diff"]), int((d.get("mask") or {}).get("size", 0)),
                                  None if d.get("kv_from") is None else int(d["kv_from"]))

    def to_dict(self) -> dict:
        d = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale, diff=self.diff)
        if self.chunk:
            d["mask"] = dict(size=self.chunk)
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d

    def dims(self, eps: float) -> GqaDims:
        return GqaDims(self.heads, self.kv_heads, self.dim, self.vdim, 0, self.scale, eps, norm=False, chunk=self.chunk, maps=2, diff=self.diff, own=self.kv_from is None)

    def validate(self, where: str) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads:
            raise InvalidArgument(f"{where}: sizes must be positive and heads a multiple of kv_heads")
        if not self.scale > 0 or self.chunk < 0:
            raise InvalidArgument(f"{where}: scale must be positive, the chunk size not negative")

    def tensor_shapes(self, width: int) -> Dict[str, Tuple[int, ...]]:
        out = {"q": (self.heads * 2 * self.dim, width), "o": (width, self.heads * self.vdim), **{k: (self.dim,) for k in ("lq1", "lk1", "lq2", "lk2")}}
        if self.kv_from is None:
            out.update({"k": (self.kv_heads * 2 * self.dim, width), "v": (self.kv_heads * self.vdim, width)})
        return out


@dataclass
class GatedLatentConfig:
    """Latent attention without positions, its heads gated."""
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_dim: int = 0
    rope_base: float = 0.0
    gate = GATE_HEAD

    @classmethod
    def from_dict(cls, d: dict) -> "GatedLatentConfig":
        return cls(int(d["heads"]), int(d["dim"]), int(d["vdim"]), int(d["kv_rank"]), float(d["scale"]))

    def to_dict(self) -> dict:
        return dict(heads=self.heads, dim=self.dim, vdim=self.vdim, kv_rank=self.kv_rank, scale=self.scale)

    def dims(self, eps: float) -> LatentDims:
        return LatentDims(self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank, self.scale, eps, gate=self.gate)

    def validate(self, where: str) -> None:
        if min(self.heads, self.dim, self.vdim, self.kv_rank) < 1 or not self.scale > 0:
            raise InvalidArgument(f"{where}: sizes and scale must be positive")

    def tensor_shapes(self, width: int) -> Dict[str, Tuple[int, ...]]:
        gates = self.heads * (self.vdim if self.gate == GATE_ELEMENT else 1)
        return {"q": (self.heads * (self.dim + self.rot_dim), width), "dkv": (self.kv_rank + self.rot_dim, width), "dkv.norm": (self.kv_rank,),
                "uk": (self.heads * self.dim, self.kv_rank), "uv": (self.heads * self.vdim, self.kv_rank), "g": (gates, width), "o": (width, self.heads * self.vdim)}


@dataclass
class RotaryGatedLatentConfig(GatedLatentConfig):
    """Latent attention with a rotated part that all heads' keys share, the elements of its heads gated."""
    gate = GATE_ELEMENT

    @classmethod
    def from_dict(cls, d: dict) -> "RotaryGatedLatentConfig":
        rot = d["rot"]
        if int(rot["dims"]) != int(d["rot_dim"]):
            raise InvalidArgument(f"Vemepel: rot.dims ({rot['dims']}) must equal rot_dim ({d['rot_dim']})")
        return cls(int(d["heads"]), int(d["dim"]), int(d["vdim"]), int(d["kv_rank"]), float(d["scale"]), int(d["rot_dim"]), float(rot["base"]))

    def to_dict(self) -> dict:
        return dict(super().to_dict(), rot_dim=self.rot_dim, rot=dict(base=self.rope_base, dims=self.rot_dim))

    def validate(self, where: str) -> None:
        super().validate(where)
        if self.rot_dim < 2 or self.rot_dim % 2 or not self.rope_base > 0:
            raise InvalidArgument(f"{where}: rot_dim must be even and positive, rot.base positive")


Mixer = Union[DifferentialConfig, GatedLatentConfig, RotaryGatedLatentConfig]
MIXERS = {"attention": DifferentialConfig, "latent_attention": GatedLatentConfig, "latent_attention_2": RotaryGatedLatentConfig}


@dataclass
class VemepelLayer:
    mixer: Mixer
    mlp: Union[DenseConfig, MoeConfig, None] = None

    @staticmethod
    def from_dict(d: dict) -> "VemepelLayer":
        if d["type"] not in MIXERS:
            raise InvalidArgument(f"Vemepel: unknown mixer {d['type']!r}")
        f = d.get("mlp")
        if f and f.get("kind") == "dense":
            mlp = DenseConfig(int(f["ff"]))
        else:
            mlp = MoeConfig.from_dict(f) if f else None
        return VemepelLayer(MIXERS[d["type"]].from_dict(d["mixer"]), mlp)

    @property
    def type(self) -> str:
        return next(k for k, c in MIXERS.items() if type(self.mixer) is c)

    def to_dict(self) -> dict:
        return dict(type=self.type, mixer=self.mixer.to_dict(), mlp=self.mlp.to_dict() if self.mlp else None)


@dataclass
class VemepelConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    layers: List[VemepelLayer] = field(default_factory=list)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def from_dict(src) -> "VemepelConfig":
        """From a parsed ``config.json`` or its path."""
        d = src if isinstance(src, dict) else json.loads(Path(src).read_text())
        c = VemepelConfig(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["logit_scale"]), [VemepelLayer.from_dict(x) for x in d["layers"]])
        c.validate()
        return c

    def to_dict(self) -> dict:
        return dict(architecture="Vemepel", vocab=self.vocab, width=self.width, norm=dict(eps=self.eps), logit_scale=self.logit_scale, layers=[x.to_dict() for x in self.layers])

    def source(self, i: int) -> int:
        """The layer whose cache rows layer ``i`` reads."""
        f = getattr(self.layers[i].mixer, "kv_from", None)
        return i if f is None else f

    def validate(self) -> None:
        if min(self.vocab, self.width, len(self.layers)) < 1:
            raise InvalidArgument("Vemepel: vocab, width and the number of layers must be positive")
        for i, l in enumerate(self.layers):
            where, m, f = f"Vemepel: layer {i}", l.mixer, l.mlp
            m.validate(where)
            if getattr(m, "kv_from", None) is not None:
                j = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if not isinstance(j, DifferentialConfig) or j.kv_from is not None or (j.kv_heads, j.dim, j.vdim) != (m.kv_heads, m.dim, m.vdim):
                    raise InvalidArgument(f"{where}: kv_from must name an earlier attention layer with keys and values of its own and the same kv_heads, dim and vdim")
            if isinstance(f, DenseConfig) and f.ff < 1:
                raise InvalidArgument(f"{where}: mlp.ff must be positive")
            if isinstance(f, MoeConfig):
                if not 1 <= f.top <= min(f.experts, MAX_TOP) or f.expert.ff < 1:
                    raise InvalidArgument(f"{where}: router.top must be between 1 and router.experts (at most {MAX_TOP}), the experts' size positive")
                if f.groups or f.shared or f.scale != 1.0 or math.isfinite(f.expert.limit):
                    raise InvalidArgument(f"{where}: the router has no groups and no scale, experts have no limit and no shared one beside them")

    @staticmethod
    def pattern(kinds: str, vocab: int, width: int, attention: dict, latent: dict, rotary: dict, mlp: Union[DenseConfig, MoeConfig, None], dense_ff: int = 0, logit_scale: float = 1.0,
                eps: float = 1e-5) -> "VemepelConfig":
        """Layers by letter: ``a`` (attention), ``s`` (attention on the keys and values of the ``a`` before it), ``l`` (latent attention without positions), ``r`` (with a rotated
        part), each kind with the sizes of its dictionary (as in ``config.json``) and all with the same feed-forward, but for dense ones of ``dense_ff`` neurons (0: none) in
        every second layer from the first on."""
        layers = []
        for i, k in enumerate(kinds):
            f = DenseConfig(dense_ff) if dense_ff and i % 2 == 0 else mlp
            m = {"a": attention, "s": attention, "l": latent, "r": rotary}[k]
            if k == "s":
                m = dict(m, kv_from=kinds.rindex("a", 0, i))
            layers.append(VemepelLayer(MIXERS[{"l": "latent_attention", "r": "latent_attention_2"}.get(k, "attention")].from_dict(m), f))
        c = VemepelConfig(vocab, width, eps, logit_scale, layers)
        c.validate()
        return c

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        W = self.width
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab, W), "head": (self.vocab, W), "final.norm": (W,)}
        for i, l in enumerate(self.layers):
            p, f = f"l{i}.", l.mlp
            out.update({p + "norm1": (W,), p + "norm1b": (W,), p + "shift": (W,), p + "dwa": (i + 2,)})
            out.update({f"{p}mix.{k}": s for k, s in l.mixer.tensor_shapes(W).items()})
            q = p + "mlp."
            if f:
                out.update({p + "norm2": (W,), p + "norm2b": (W,)})
            if isinstance(f, DenseConfig):
                out.update({q + "up": (f.ff, W), q + "down": (W, f.ff), q + "act": (4,)})
            elif f:
                out.update({q + "router": (f.experts, W), q + "router.b": (f.experts,)})
                for e in range(f.experts):
                    out.update({f"{q}e{e}.gate": (f.expert.ff, W), f"{q}e{e}.up": (f.expert.ff, W), f"{q}e{e}.down": (W, f.expert.ff)})
        return out

    @property
    def optional_tensors(self) -> List[str]:
        """Norms of the feed-forward that a layer does not have: ignored."""
        return [f"l{i}.{n}" for i, l in enumerate(self.layers) if l.mlp is None for n in ("norm2", "norm2b")]


class RandomVemepelWeights:
    """Random weights made tensor by tensor when they are asked for (large configurations never exist twice in memory)."""

    def __init__(self, cfg: VemepelConfig, device="cuda", seed: int = 0):
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
        if name.endswith("dkv.norm"):
            t = 1.0 + 0.05 * t
        elif name.endswith(".shift"):
            t = torch.sigmoid(t)
        elif name.endswith(".dwa"):
            t = 0.1 * t
            t[-1] += 1.0
        elif name.endswith(".act"):
            t = 0.5 + 0.1 * t
        elif len(s) == 2 and name != "embed":
            t = t / math.sqrt(s[1])
        elif name != "embed":
            t = 0.05 * t
        return t.to(torch.bfloat16)


@dataclass
class _Layer:
    """Weights of one layer. Of ``attn`` and ``latent`` one is set, of ``dense`` and ``moe`` at most one. ``proj`` and ``out`` are the mixer's first and last product; norm
    weights include their one, ``average`` weighs the embedding output and the layers' results."""
    norm1: torch.Tensor
    norm1b: torch.Tensor
    share: torch.Tensor
    average: torch.Tensor
    proj: torch.Tensor
    out: torch.Tensor
    attn: Optional[GqaWeights] = None
    latent: Optional[LatentWeights] = None
    source: int = 0                      # the layer whose cache rows the mixer reads
    norm2: Optional[torch.Tensor] = None
    norm2b: Optional[torch.Tensor] = None
    dense: Optional[DensePolyWeights] = None
    moe: Optional[MoeWeights] = None
    tables: Tuple[Optional[torch.Tensor], Optional[torch.Tensor]] = (None, None)
    buffers: object = None
    mixed: Optional[torch.Tensor] = None
    g_proj: Optional[_SplitKGemm] = None
    g_out: Optional[_SplitKGemm] = None
    g_up: Optional[_SplitKGemm] = None
    g_down: Optional[_SplitKGemm] = None

    @property
    def mixer(self):
        return self.attn or self.latent


class VemepelModel:
    """Weights and layer schedule; ``weights`` maps the names of :meth:`VemepelConfig.tensor_shapes` to tensors (anything with ``[]``, ``in`` and ``keys``)."""

    def __init__(self, cfg: VemepelConfig, weights, device="cuda", dtype: torch.dtype = torch.bfloat16):
        cfg.validate()
        if dtype not in (torch.bfloat16, torch.float32):
            raise InvalidArgument("Vemepel runs in bfloat16 or float32")
        self.cfg, self.device, self.dtype, self.vocab = cfg, torch.device(device), dtype, cfg.vocab
        if self.device.type != "cuda":
            raise InvalidArgument("Vemepel runs on a CUDA device (its operators are CUDA kernels)")
        self._load(weights)

    # -- weights ---------------------------------------------------------------
    def _load(self, weights) -> None:
        cfg, dev, dt, W = self.cfg, self.device, self.dtype, self.cfg.width
        get = checked_weights("Vemepel", cfg.tensor_shapes(), weights, dev, cfg.optional_tensors)

        def matrix(t):
            m = torch.zeros(t.shape[0], round_up(t.shape[1], 32), device=dev, dtype=dt)
            m[:, : t.shape[1]] = t
            return m[:, : t.shape[1]]

        def norm(name, scale=1.0):
            return padded_vector((1.0 + get(name).float()) * scale, dev)
        self.embed, self.head = matrix(get("embed")), matrix(get("head"))
        self.final_norm = norm("final.norm", cfg.logit_scale)           # the logits' factor rides on their operand
        self.layers: List[_Layer] = []
        for i, l in enumerate(cfg.layers):
            p, m, f = f"l{i}.", l.mixer, l.mlp
            q, D = p + "mix.", m.dims(cfg.eps)
            mix = {k: get(q + k) for k in m.tensor_shapes(W)}
            vectors = (norm(p + "norm1"), norm(p + "norm1b"), padded_vector(get(p + "shift"), dev), get(p + "dwa").to(dev, torch.float32).contiguous())
            if isinstance(m, DifferentialConfig):
                rows = [pack_head_rows(mix["q"], 2 * m.heads, m.dim, dev, dt)]
                if D.own:
                    rows += [pack_head_rows(mix["k"], 2 * m.kv_heads, m.dim, dev, dt), pack_head_rows(mix["v"], m.kv_heads, m.vdim, dev, dt)]
                w = GqaWeights.pack(D, None, None, dev, blend=differential_blend(*(mix[k] for k in ("lq1", "lk1", "lq2", "lk2")), m.diff))
                layer = _Layer(*vectors, matrix(torch.cat(rows)), matrix(pack_head_columns(mix["o"], m.heads, m.vdim, dev, dt)), attn=w)
            else:
                w = LatentWeights.pack(D, *(mix[k] for k in ("q", "dkv", "dkv.norm", "uk", "uv", "o")), dev, dt, gate=mix["g"])
                layer = _Layer(*vectors, w.proj, w.out, latent=w)
            layer.source = cfg.source(i)
            q = p + "mlp."
            if f:
                layer.norm2, layer.norm2b = norm(p + "norm2"), norm(p + "norm2b")
            if isinstance(f, DenseConfig):
                layer.dense = DensePolyWeights.pack(get(q + "up"), get(q + "down"), get(q + "act"), cfg.eps, dev, dt)
            elif f:
                stack = ExpertStack.pack(*([get(f"{q}e{e}.{k}") for e in range(f.experts)] for k in ("gate", "up", "down")), f.expert.limit, dev, dt)
                layer.moe = MoeWeights(matrix(get(q + "router")), stack, None, W, f.top, form=ACTIVATION, rule=RouteRule(padded_vector(get(q + "router.b"), dev), softmax=True))
            self.layers.append(layer)
        self._ld = round_up(W, 8)

    @property
    def cache_rows(self) -> List[int]:
        return [l.mixer.dims.row if l.mixer.dims.own else 0 for l in self.layers]

    @property
    def state_sizes(self) -> List[int]:
        return [round_up(self.cfg.width, 4)] * len(self.layers)

    def prepare(self, max_positions: int) -> None:
        """Rotation tables for positions below ``max_positions``."""
        made: dict = {}
        for l, c in zip(self.layers, self.cfg.layers):
            if l.latent and l.latent.dims.rot_dim:
                key = (c.mixer.rot_dim, c.mixer.rope_base)
                if key not in made:
                    made[key] = rotary_pair_tables(max_positions, *key, self.device)
                l.tables = made[key]

    def _next_norm(self, i: int) -> torch.Tensor:
        """Norm weights of layer ``i``'s operand; past the last layer the model's norm."""
        return self.layers[i].norm1 if i < len(self.layers) else self.final_norm

    def _shift(self, i: int, cache) -> Optional[TokenShift]:
        return TokenShift(self.layers[i].share, cache.states.data[i]) if i < len(self.layers) else None

    # -- prompts and any ragged batch ------------------------------------------
    def _mix_rows(self, h: torch.Tensor, l: _Layer, batch, cache) -> SublayerOutput:
        if l.latent:
            return latent_attention_rows(h, l.latent, batch, cache.rows[l.source], *l.tables)
        a = torch.empty(h.shape[0], l.out.shape[1], device=h.device, dtype=h.dtype)
        gqa_attention_rows(linear_rows(h, l.proj), l.attn, batch, cache.rows[l.source], *l.tables, None, a)
        y = linear_rows(a, l.out, out_f32=True)
        return SublayerOutput(planes=y.as_strided((1, y.shape[0], y.shape[1]), (0, y.stride(0), 1)))

    @torch.no_grad()
    def forward_rows(self, batch, cache, taps: Optional[list] = None) -> Optional[torch.Tensor]:
        """Runs the new tokens of a :class:`RowBatch`, writes their cache rows, advances the states and returns the logits of ``batch.want`` (``None`` if empty). ``taps``
        collects what every layer hands on, ``[rows, width]``."""
        T, W, eps, n = batch.rows, self.cfg.width, self.cfg.eps, len(self.layers)
        streams = torch.empty(n + 2, T, self._ld, device=self.device, dtype=torch.float32)
        x, results = streams[0], streams[1:]                # the residual; the embedding output and every layer's result
        h = torch.empty(T, self._ld, device=self.device, dtype=self.dtype)[:, :W]
        rstd = torch.empty(T, device=self.device, dtype=torch.float32)
        spans = batch.memory_plan(0).spans
        depth_embed(batch.ids, self.embed, x, results, None, eps, T, rstd=rstd)
        for i, l in enumerate(self.layers):
            token_shift(x, rstd, l.norm1, self._shift(i, cache), spans, batch.seq_of, h, T, W)
            y, w = self._mix_rows(h, l, batch, cache), l.norm1b
            if l.norm2 is not None:
                residual_update(x, y, w, eps, h, T, W, l.norm2)
                y, w = dense_poly_rows(h, l.dense) if l.dense else moe_rows(h, l.moe), l.norm2b
            last = i + 1 == n
            depth_update(x, results, l.average, y, w, self._next_norm(i + 1), eps, self.dtype, T, W, h=h if last else None, rstd=None if last else rstd,
                         store=not last or taps is not None)
            if taps is not None:
                taps.append(x[:, :W].clone())
        if batch.want is None:
            return None
        hw = torch.empty(batch.want.numel(), self._ld, device=self.device, dtype=self.dtype)[:, :W]
        hw.copy_(h[batch.want])
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
                rows[n] = torch.zeros(PAD_ROWS, round_up(n, 8), device=dev, dtype=self.dtype)
            return rows[n][:, :n]
        for l in self.layers:
            D = l.mixer.dims
            if D not in shared:
                shared[D] = (GqaDecodeBuffers if l.attn else LatentDecodeBuffers)(D, max_batch, max_tokens, dev)
            l.buffers = shared[D]
            if l.attn:
                l.mixed = row_buffer(D.out_cols)
            l.g_proj, l.g_out = _SplitKGemm(l.proj, dev, planes), _SplitKGemm(l.out, dev, planes)
            if l.dense:
                l.g_up, l.g_down = _SplitKGemm(l.dense.up, dev, planes), _SplitKGemm(l.dense.down, dev, planes)
        self._g_head = _SplitKGemm(self.head, dev)
        moes = [l.moe for l in self.layers if l.moe]
        self._moe_buffers = MoeSmallBuffers.allocate(moes, dev) if moes else None
        self._act = {n: row_buffer(n) for n in {l.dense.ff for l in self.layers if l.dense}}
        self._results = torch.zeros(len(self.layers) + 1, PAD_ROWS, self._ld, device=dev)
        self._x = torch.zeros(PAD_ROWS, self._ld, device=dev)
        self._h = torch.zeros(PAD_ROWS, self._ld, device=dev, dtype=self.dtype)[:, :W]
        self._logits = torch.zeros(PAD_ROWS, round_up(self.vocab, 4), device=dev)[:, : self.vocab]

    def _mix_decode(self, l: _Layer, state, B: int, cache) -> SublayerOutput:
        g = l.g_proj
        g(self._h)
        if l.attn:
            a = l.mixed
            gqa_attention_decode(g.planes, g.splits, l.attn, l.buffers, state, cache.rows[l.source], *l.tables, B, 0, a)
        else:
            a = latent_attention_decode(g.planes, g.splits, l.latent, l.buffers, state, cache.rows[l.source], *l.tables, B)
        l.g_out(a)
        return SublayerOutput(planes=l.g_out.planes)

    def _feed_decode(self, l: _Layer, B: int) -> SublayerOutput:
        if l.moe:
            return moe_small(self._h, l.moe, self._moe_buffers, B)
        a = self._act[l.dense.ff]
        l.g_up(self._h)
        poly_norm_planes(l.g_up.planes, l.g_up.splits, B, l.dense.coef, l.dense.eps, a)
        l.g_down(a)
        return SublayerOutput(planes=l.g_down.planes)

    @torch.no_grad()
    def decode(self, state, B: int, cache) -> torch.Tensor:
        """One token for the first ``B`` sequences of ``state``; returns the logits buffer ``[16, vocab]`` (rows below ``B`` are valid)."""
        W, eps, x, h, results, n = self.cfg.width, self.cfg.eps, self._x, self._h, self._results, len(self.layers)
        where = dict(slots=state.slots, positions=state.positions)
        depth_embed(state.tokens, self.embed, x, results, self._next_norm(0), eps, B, h, shift=self._shift(0, cache), **where)
        for i, l in enumerate(self.layers):
            y, w = self._mix_decode(l, state, B, cache), l.norm1b
            if l.norm2 is not None:
                residual_update(x, y, w, eps, h, B, W, l.norm2)
                y, w = self._feed_decode(l, B), l.norm2b
            depth_update(x, results, l.average, y, w, self._next_norm(i + 1), eps, self.dtype, B, W, h, shift=self._shift(i + 1, cache), store=i + 1 < n, **where)
        self._g_head(h)
        g = self._g_head
        _lib.call("ft_splitk_reduce", g.planes, g.splits, B, self.vocab, g.ldp, g.plane_stride, None, self._logits, self._logits.stride(0), 1, _lib.S())
        return self._logits
