"""Pufevik: a decoder whose layers are either full attention with values mixed from the first such layer, or a windowed attention and a matrix memory side by side, each
followed by a dense gated feed-forward; one residual, with the norm on every sublayer's output.

``config.json`` carries a list of layers, each with its own mixer and feed-forward sizes; tensors are named ``l<i>.mix.*`` (``l<i>.mix.left.*`` and ``l<i>.mix.right.*``
where two mixers run side by side), ``l<i>.mlp.*``, ``l<i>.norm1`` and ``l<i>.norm2`` (see :meth:`PufevikConfig.tensor_shapes`). The model runs inside
:class:`~ferrotorch_b200.models.serving.ServingEngine`:

* prompts (any ragged batch): one tcgen05 GEMM for all projections of a mixer (a second, small one with f32 results for its gates), ragged flash attention over the
  pages, the chunked walk of the matrix memory, one GEMM for both mixers' outputs, one pass over the residual per sublayer;
* decode (bf16, up to 16 sequences): split-K weight streaming, whose partial sums every kernel behind it consumes directly -- nine or ten launches a layer, replayed from
  one CUDA graph;
* f32: the same structure on exact FMA-pipe products, a plain attention kernel and the matrix memory token by token.
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
from ..ops.gqa_attention import (GATE_ELEMENT, GATE_HEAD, GqaDecodeBuffers, GqaDims, GqaWeights, gqa_attention_decode, gqa_attention_rows, pack_head_columns, pack_head_rows)
from ..ops.latent_attention import rotary_pair_tables
from ..ops.matrix_memory import MemoryDims, MemoryWeights, matrix_memory_decode, matrix_memory_rows
from ..ops.moe import linear_rows
from ..ops.residual import DenseGatedWeights, dense_gated_rows, gated_act_planes, residual_embed, residual_update
from ..ops.streams import SublayerOutput, padded_vector, round_up
from .llama_infer import PAD_ROWS, _SplitKGemm
from .registry import checked_weights

ACTIVATION = "gelu_tanh"             # fixed by the design


@dataclass
class AttentionConfig:
    """Grouped-query attention; ``window`` 0 means every earlier position, ``keep_first`` tokens stay visible beside a window; ``scaling``: YaRN scaling of the rotation (``factor``,
    ``original``, ``fast``, ``slow``)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int = 0
    rope_base: float = 10000.0
    window: int = 0
    v_mix: bool = False
    keep_first: int = 0
    scaling: Optional[Dict[str, float]] = None

    @staticmethod
    def from_dict(d: dict) -> "AttentionConfig":
        rot, mask = d.get("rot") or {}, d.get("mask") or {}
        s = rot.get("scaling")
        return AttentionConfig(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]), int(rot.get("dims", 0)), float(rot.get("base", 10000.0)),
                               int(mask.get("size", 0)), bool(d.get("v_mix", False)), int(mask.get("keep_first", 0)),
                               {k: float(s[k]) for k in ("factor", "original", "fast", "slow")} if s else None)

    def to_dict(self) -> dict:
        d = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale, rot=dict(base=self.rope_base, dims=self.rot_dims))
        if self.scaling:
            d["rot"]["scaling"] = dict(self.scaling)
        if self.window:
            d["mask"] = dict(size=self.window)
            if self.keep_first:
                d["mask"]["keep_first"] = self.keep_first
        if self.v_mix:
            d["v_mix"] = True
        return d

    def validate(self, where: str) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads:
            raise InvalidArgument(f"{where}: sizes must be positive and heads a multiple of kv_heads")
        if self.rot_dims < 0 or self.rot_dims % 2 or self.rot_dims > self.dim or not self.rope_base > 0:
            raise InvalidArgument(f"{where}: rot.dims must be even and at most dim, rot.base positive")
        if not self.scale > 0 or self.window < 0 or self.keep_first < 0:
            raise InvalidArgument(f"{where}: scale must be positive, the window and the number of kept tokens not negative")
        if self.scaling and not (min(self.scaling.values()) > 0 and self.rope_base != 1.0):
            raise InvalidArgument(f"{where}: the constants of rot.scaling must be positive")

    @property
    def rope_scaling(self) -> Optional[dict]:
        """The scaling in the form of :func:`~ferrotorch_b200.ops.llama.rope_inv_freq`."""
        s = self.scaling
        return s and dict(type="yarn", factor=s["factor"], original_max_position=s["original"], beta_fast=s["fast"], beta_slow=s["slow"],
                          attention_factor=0.1 * math.log(s["factor"]) + 1.0)


@dataclass
class MemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @staticmethod
    def from_dict(d: dict) -> "MemoryConfig":
        return MemoryConfig(int(d["heads"]), int(d["dim"]), int(d["vdim"]), float(d["gate_cap"]))

    def to_dict(self) -> dict:
        return dict(heads=self.heads, dim=self.dim, vdim=self.vdim, gate_cap=self.gate_cap)

    def validate(self, where: str) -> None:
        if min(self.heads, self.dim, self.vdim) < 1 or not self.gate_cap > 0:
            raise InvalidArgument(f"{where}: sizes and gate_cap must be positive")


@dataclass
class ParallelConfig:
    """An attention and a matrix memory that read the same input; their outputs are added with the two scales."""
    left: AttentionConfig
    right: MemoryConfig
    left_scale: float = 1.0
    right_scale: float = 1.0

    @staticmethod
    def from_dict(d: dict) -> "ParallelConfig":
        return ParallelConfig(AttentionConfig.from_dict(d["left"]), MemoryConfig.from_dict(d["right"]), float(d["left_scale"]), float(d["right_scale"]))

    def to_dict(self) -> dict:
        return dict(left=self.left.to_dict(), right=self.right.to_dict(), left_scale=self.left_scale, right_scale=self.right_scale)

    def validate(self, where: str) -> None:
        self.left.validate(where + " left")
        self.right.validate(where + " right")
        if self.left.v_mix:
            raise InvalidArgument(f"{where} left: values are mixed in 'attention' layers only")


@dataclass
class PufevikLayer:
    mixer: Union[AttentionConfig, ParallelConfig]
    ff: int = 0                      # neurons of the feed-forward, 0: none

    @staticmethod
    def from_dict(d: dict) -> "PufevikLayer":
        kinds = {"attention": AttentionConfig, "parallel": ParallelConfig}
        if d["type"] not in kinds:
            raise InvalidArgument(f"Pufevik: unknown mixer {d['type']!r}")
        mlp = d.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise InvalidArgument(f"Pufevik: unknown feed-forward kind {mlp['kind']!r}")
        if mlp and int(mlp["ff"]) < 1:
            raise InvalidArgument("Pufevik: mlp.ff must be positive")
        return PufevikLayer(kinds[d["type"]].from_dict(d["mixer"]), int(mlp["ff"]) if mlp else 0)

    def to_dict(self) -> dict:
        return dict(type="parallel" if isinstance(self.mixer, ParallelConfig) else "attention", mixer=self.mixer.to_dict(), mlp=dict(kind="dense", ff=self.ff) if self.ff else None)


@dataclass
class PufevikConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: List[PufevikLayer] = field(default_factory=list)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def from_dict(src) -> "PufevikConfig":
        """From a parsed ``config.json`` or its path."""
        d = src if isinstance(src, dict) else json.loads(Path(src).read_text())
        c = PufevikConfig(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["embedding"]["scale"]), [PufevikLayer.from_dict(x) for x in d["layers"]])
        c.validate()
        return c

    def to_dict(self) -> dict:
        return dict(architecture="Pufevik", vocab=self.vocab, width=self.width, norm=dict(eps=self.eps), embedding=dict(scale=self.embedding_scale),
                    layers=[x.to_dict() for x in self.layers])

    @property
    def mixing_layers(self) -> List[int]:
        """Layers that mix values; the first of them supplies the values the others mix in."""
        return [i for i, l in enumerate(self.layers) if isinstance(l.mixer, AttentionConfig) and l.mixer.v_mix]

    def validate(self) -> None:
        if min(self.vocab, self.width, len(self.layers)) < 1:
            raise InvalidArgument("Pufevik: vocab, width and the number of layers must be positive")
        for i, l in enumerate(self.layers):
            l.mixer.validate(f"Pufevik: layer {i}")
            a = l.mixer if isinstance(l.mixer, AttentionConfig) else l.mixer.left
            if a is l.mixer and a.window:
                raise InvalidArgument(f"Pufevik: layer {i}: a window stands in the left half of 'parallel' layers only")
            if a.keep_first or a.scaling:
                raise InvalidArgument(f"Pufevik: layer {i}: no kept first tokens, no scaled rotation")
        mix = [self.layers[i].mixer for i in self.mixing_layers]
        if any((m.kv_heads, m.vdim) != (mix[0].kv_heads, mix[0].vdim) for m in mix):
            raise InvalidArgument("Pufevik: layers that mix values must have the same kv_heads and vdim")

    @staticmethod
    def pattern(kinds: str, vocab: int, width: int, ff: int, heads: int, kv_heads: int, dim: int, vdim: int, window: int, memory_heads: int, memory_dim: int, memory_vdim: int,
                gate_cap: float = 15.0, rope_base: float = 10000.0, eps: float = 1e-6) -> "PufevikConfig":
        """Layers by letter: ``p`` (attention and memory side by side) or ``a`` (full attention), all of the same sizes."""
        att = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5, rot_dims=dim // 2 // 2 * 2, rope_base=rope_base)

        def layer(k):
            if k == "a":
                return PufevikLayer(AttentionConfig(**att, v_mix=True), ff)
            return PufevikLayer(ParallelConfig(AttentionConfig(**att, window=window), MemoryConfig(memory_heads, memory_dim, memory_vdim, gate_cap)), ff)
        c = PufevikConfig(vocab, width, eps, math.sqrt(width), [layer(k) for k in kinds])
        c.validate()
        return c

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        W = self.width
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab, W), "head": (self.vocab, W), "final.norm": (W,)}
        for i, l in enumerate(self.layers):
            p, m = f"l{i}.", l.mixer
            out[p + "norm1"] = (W,)

            def attention(q, a, whole, gate_rows):
                out.update({q + "q": (a.heads * a.dim, W), q + "k": (a.kv_heads * a.dim, W), q + "v": (a.kv_heads * a.vdim, W), q + "g": (gate_rows, W),
                            q + "o": (W, a.heads * a.vdim), q + "q.norm": (a.heads * a.dim if whole else a.dim,), q + "k.norm": (a.kv_heads * a.dim if whole else a.dim,)})
            if isinstance(m, AttentionConfig):
                attention(p + "mix.", m, False, m.heads * m.vdim)
                if m.v_mix:
                    out[p + "mix.vmix"] = ()
            else:
                attention(p + "mix.left.", m.left, True, m.left.heads)
                out[p + "mix.left.sink"] = (m.left.heads,)
                r, q = m.right, p + "mix.right."
                out.update({q + "q": (r.heads * r.dim, W), q + "k": (r.heads * r.dim, W), q + "v": (r.heads * r.vdim, W), q + "g": (r.heads * r.vdim, W),
                            q + "o": (W, r.heads * r.vdim), q + "norm": (r.heads * r.vdim,)})
                for g in "if":
                    out.update({q + g: (r.heads, W), f"{q}{g}.b": (r.heads,)})
            if l.ff:
                out.update({p + "norm2": (W,), p + "mlp.gate": (l.ff, W), p + "mlp.up": (l.ff, W), p + "mlp.down": (W, l.ff)})
        return out

    @property
    def optional_tensors(self) -> List[str]:
        """Mixing weights that nothing reads: the first mixing layer's own, and those of layers that do not mix."""
        later = self.mixing_layers[1:]
        return [f"l{i}.mix.vmix" for i, l in enumerate(self.layers) if isinstance(l.mixer, AttentionConfig) and i not in later]


class RandomPufevikWeights:
    """Random weights made tensor by tensor when they are asked for (large configurations never exist twice in memory)."""

    def __init__(self, cfg: PufevikConfig, device="cuda", seed: int = 0):
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
        if name.endswith(".vmix"):
            t = 0.5 + 0.1 * t
        elif name.endswith(("norm", "norm1", "norm2")):
            t = 1.0 + 0.05 * t
        elif name.endswith(".f.b"):
            t = 3.0 + t
        elif len(s) == 2:
            t = t / math.sqrt(s[1])
        return t.to(torch.bfloat16)


@dataclass
class _Mixer:
    """Weights of one layer's mixer. ``proj`` ``[columns, width]``: queries, keys, values (and, with an element gate, its rows) of the attention, then the matrix memory's
    projections, then from row ``main`` on the gates whose pre-activations stay in f32 (heads of the attention, input and forget gates). ``out`` takes the attention's
    and the memory's outputs side by side."""
    attn: GqaWeights
    memory: Optional[MemoryWeights]
    proj: torch.Tensor
    main: int
    out: torch.Tensor
    keeps_values: bool = False
    g_proj: Optional[_SplitKGemm] = None
    g_out: Optional[_SplitKGemm] = None
    tables: Tuple[torch.Tensor, torch.Tensor] = None
    buffers: Optional[GqaDecodeBuffers] = None

    @property
    def out_cols(self) -> int:
        return self.out.shape[1]

    @property
    def memory_col(self) -> int:
        return self.attn.dims.qkv_cols

    @property
    def memory_gate_col(self) -> int:
        return self.main + round_up(self.attn.dims.heads, 8)


@dataclass
class _Sub:
    """One sublayer: exactly one of ``mixer`` and ``ff``, and the weight of the norm on its output."""
    layer: int
    norm: torch.Tensor
    mixer: Optional[_Mixer] = None
    ff: Optional[DenseGatedWeights] = None
    g_gu: Optional[_SplitKGemm] = None
    g_down: Optional[_SplitKGemm] = None
    last_of_layer: bool = False


class PufevikModel:
    """Weights and layer schedule; ``weights`` maps the names of :meth:`PufevikConfig.tensor_shapes` to tensors (anything with ``[]``, ``in`` and ``keys``)."""

    def __init__(self, cfg: PufevikConfig, weights, device="cuda", dtype: torch.dtype = torch.bfloat16):
        cfg.validate()
        if dtype not in (torch.bfloat16, torch.float32):
            raise InvalidArgument("Pufevik runs in bfloat16 or float32")
        self.cfg, self.device, self.dtype, self.vocab = cfg, torch.device(device), dtype, cfg.vocab
        if self.device.type != "cuda":
            raise InvalidArgument("Pufevik runs on a CUDA device (its operators are CUDA kernels)")
        self._load(weights)

    # -- weights ---------------------------------------------------------------
    def _load(self, weights) -> None:
        cfg, dev, dt, W = self.cfg, self.device, self.dtype, self.cfg.width
        get = checked_weights("Pufevik", cfg.tensor_shapes(), weights, dev, cfg.optional_tensors)

        def matrix(t):
            m = torch.zeros(t.shape[0], round_up(t.shape[1], 32), device=dev, dtype=dt)
            m[:, : t.shape[1]] = t
            return m[:, : t.shape[1]]

        def padded_rows(t, rows):
            out = torch.zeros(rows, t.shape[1], device=dev, dtype=dt)
            out[: t.shape[0]] = t
            return out

        def qkv(p, a):
            return [pack_head_rows(get(p + "q"), a.heads, a.dim, dev, dt), pack_head_rows(get(p + "k"), a.kv_heads, a.dim, dev, dt),
                    pack_head_rows(get(p + "v"), a.kv_heads, a.vdim, dev, dt)]
        mixing = cfg.mixing_layers
        self.embed, self.head = matrix(get("embed")), matrix(get("head"))
        self.final_norm = padded_vector(get("final.norm"), dev)
        self.subs: List[_Sub] = []
        for i, l in enumerate(cfg.layers):
            p, m = f"l{i}.", l.mixer
            a = m if isinstance(m, AttentionConfig) else m.left
            sizes = (a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dims, a.scale, cfg.eps)
            if a is m:
                q = p + "mix."
                dims = GqaDims(*sizes, gate=GATE_ELEMENT)
                aw = GqaWeights.pack(dims, get(q + "q.norm"), get(q + "k.norm"), dev, mix=get(q + "vmix") if i in mixing[1:] else None)
                rows = qkv(q, a) + [pack_head_rows(get(q + "g"), a.heads, a.vdim, dev, dt)]
                proj = matrix(torch.cat(rows))
                mixer = _Mixer(aw, None, proj, proj.shape[0], matrix(pack_head_columns(get(q + "o"), a.heads, a.vdim, dev, dt)), keeps_values=i in mixing[:1])
            else:
                q, s, r = p + "mix.left.", p + "mix.right.", m.right
                dims = GqaDims(*sizes, window=a.window, whole_norm=True, gate=GATE_HEAD, out_scale=m.left_scale)
                aw = GqaWeights.pack(dims, get(q + "q.norm"), get(q + "k.norm"), dev, sink=get(q + "sink"))
                md = MemoryDims(r.heads, r.dim, r.vdim, r.gate_cap, cfg.eps, m.right_scale)
                mw = MemoryWeights.pack(md, get(s + "i.b"), get(s + "f.b"), get(s + "norm"), dev)
                rows = qkv(q, a) + [pack_head_rows(get(s + k), r.heads, n, dev, dt) for k, n in (("q", r.dim), ("k", r.dim), ("v", r.vdim), ("g", r.vdim))]
                main = sum(t.shape[0] for t in rows)
                rows += [padded_rows(get(q + "g"), round_up(a.heads, 8)), padded_rows(get(s + "i"), md.h8), padded_rows(get(s + "f"), md.h8)]
                outs = [pack_head_columns(get(q + "o"), a.heads, a.vdim, dev, dt), pack_head_columns(get(s + "o"), r.heads, r.vdim, dev, dt)]
                mixer = _Mixer(aw, mw, matrix(torch.cat(rows)), main, matrix(torch.cat(outs, 1)))
            self.subs.append(_Sub(i, padded_vector(get(p + "norm1"), dev), mixer=mixer))
            if l.ff:
                ff = DenseGatedWeights.pack(get(p + "mlp.gate"), get(p + "mlp.up"), get(p + "mlp.down"), dev, dt, ACTIVATION)
                self.subs.append(_Sub(i, padded_vector(get(p + "norm2"), dev), ff=ff))
            self.subs[-1].last_of_layer = True
        self._ld = round_up(W, 8)

    @property
    def mixers(self) -> List[_Mixer]:
        return [s.mixer for s in self.subs if s.mixer]

    @property
    def cache_rows(self) -> List[int]:
        return [m.attn.dims.row for m in self.mixers]

    @property
    def state_sizes(self) -> List[int]:
        return [m.memory.dims.state_size if m.memory else 0 for m in self.mixers]

    def prepare(self, max_positions: int) -> None:
        """Rotation tables for positions below ``max_positions``."""
        made: dict = {}
        for s in self.subs:
            if s.mixer:
                m = self.cfg.layers[s.layer].mixer
                a = m if isinstance(m, AttentionConfig) else m.left
                key = (a.rot_dims, a.rope_base)
                if key not in made:
                    made[key] = rotary_pair_tables(max_positions, a.rot_dims, a.rope_base, self.device)
                s.mixer.tables = made[key]

    # -- prompts and any ragged batch ------------------------------------------
    def _mix_rows(self, h: torch.Tensor, layer: int, m: _Mixer, batch, cache, carry: dict) -> SublayerOutput:
        D = m.attn.dims
        x = linear_rows(h, m.proj[: m.main])
        gates = linear_rows(h, m.proj[m.main:], out_f32=True) if m.memory else None
        a = torch.empty(h.shape[0], m.out_cols, device=h.device, dtype=h.dtype)
        first = carry.get("values") if m.attn.mix is not None else None
        gqa_attention_rows(x, m.attn, batch, cache.rows[layer], *m.tables, gates[:, : D.heads] if m.memory else x[:, D.qkv_cols:], a[:, : D.out_cols], first)
        if m.keeps_values:
            carry["values"] = x[:, D.v_col: D.qkv_cols]
        if m.memory:
            matrix_memory_rows(x[:, m.memory_col:], gates[:, m.memory_gate_col - m.main:], m.memory, batch, cache.states.data[layer], a[:, D.out_cols:])
        y = linear_rows(a, m.out, out_f32=True)
        return SublayerOutput(planes=y.as_strided((1, y.shape[0], y.shape[1]), (0, y.stride(0), 1)))

    @torch.no_grad()
    def forward_rows(self, batch, cache, taps: Optional[list] = None) -> Optional[torch.Tensor]:
        """Runs the new tokens of a :class:`RowBatch`, writes their cache rows, advances the states and returns the logits of ``batch.want`` (``None`` if empty). ``taps``
        collects the residual after every layer, ``[rows, width]``."""
        cfg, T, W = self.cfg, batch.rows, self.cfg.width
        x = torch.empty(T, self._ld, device=self.device, dtype=torch.float32)
        h = torch.empty(T, self._ld, device=self.device, dtype=self.dtype)[:, :W]
        residual_embed(batch.ids, self.embed, cfg.embedding_scale, x, h, T)
        carry: dict = {}
        for k, s in enumerate(self.subs):
            y = self._mix_rows(h, s.layer, s.mixer, batch, cache, carry) if s.mixer else dense_gated_rows(h, s.ff)
            last = k + 1 == len(self.subs)
            residual_update(x, y, s.norm, cfg.eps, h, T, W, self.final_norm if last else None, store=not last or taps is not None)
            if taps is not None and s.last_of_layer:
                taps.append(x[:, :W].clone())
        if batch.want is None:
            return None
        hw = torch.empty(batch.want.numel(), self._ld, device=self.device, dtype=self.dtype)[:, :W]
        hw.copy_(h[batch.want])
        return linear_rows(hw, self.head, out_f32=True)

    # -- decode ------------------------------------------------------------------
    def decode_supported(self) -> bool:
        """Whether the captured decode step covers this model: bf16, and sizes within its kernels' shared memory."""
        return self.dtype == torch.bfloat16 and all(m.attn.dims.decode_supported() and (m.memory is None or m.memory.dims.decode_supported()) for m in self.mixers)

    def decode_begin(self, max_batch: int, max_tokens: int) -> None:
        """Allocates the decode step's buffers."""
        cfg, dev, W = self.cfg, self.device, self.cfg.width
        planes: dict = {}
        shared: Dict[GqaDims, GqaDecodeBuffers] = {}
        for s in self.subs:
            if s.mixer:
                m = s.mixer
                if m.attn.dims not in shared:
                    shared[m.attn.dims] = GqaDecodeBuffers(m.attn.dims, max_batch, max_tokens, dev)
                m.buffers = shared[m.attn.dims]
                m.g_proj, m.g_out = _SplitKGemm(m.proj, dev, planes), _SplitKGemm(m.out, dev, planes)
            else:
                s.g_gu, s.g_down = _SplitKGemm(s.ff.gu, dev, planes), _SplitKGemm(s.ff.down, dev, planes)
        self._g_head = _SplitKGemm(self.head, dev)
        ffs = [s.ff for s in self.subs if s.ff]
        self._x = torch.zeros(PAD_ROWS, self._ld, device=dev)
        self._h = torch.zeros(PAD_ROWS, self._ld, device=dev, dtype=self.dtype)[:, :W]
        self._mixed = [torch.zeros(PAD_ROWS, n, device=dev, dtype=self.dtype) for n in sorted({m.out_cols for m in self.mixers})]
        self._act = [torch.zeros(PAD_ROWS, n, device=dev, dtype=self.dtype) for n in sorted({f.fp for f in ffs})]
        first = next((m.attn.dims for m in self.mixers if m.keeps_values), None)
        self._values = torch.zeros(PAD_ROWS, first.kv_heads * first.v16, device=dev) if first else None
        self._logits = torch.zeros(PAD_ROWS, round_up(self.vocab, 4), device=dev)[:, : self.vocab]

    @torch.no_grad()
    def decode(self, state, B: int, cache) -> torch.Tensor:
        """One token for the first ``B`` sequences of ``state``; returns the logits buffer ``[16, vocab]`` (rows below ``B`` are valid)."""
        cfg, W, x, h = self.cfg, self.cfg.width, self._x, self._h
        mixed, act = {t.shape[1]: t for t in self._mixed}, {t.shape[1]: t for t in self._act}
        residual_embed(state.tokens, self.embed, cfg.embedding_scale, x, h, B)
        for k, s in enumerate(self.subs):
            if s.mixer:
                m, g = s.mixer, s.mixer.g_proj
                D, a = m.attn.dims, mixed[s.mixer.out_cols]
                g(h)
                gate_col = m.main if m.memory else D.qkv_cols
                gqa_attention_decode(g.planes, g.splits, m.attn, m.buffers, state, cache.rows[s.layer], *m.tables, B, gate_col, a[:, : D.out_cols],
                                     self._values if m.keeps_values else None, self._values if m.attn.mix is not None else None)
                if m.memory:
                    matrix_memory_decode(g.planes, g.splits, m.memory, state, cache.states.data[s.layer], B, m.memory_col, m.memory_gate_col, a[:, D.out_cols:])
                m.g_out(a)
                y = SublayerOutput(planes=m.g_out.planes)
            else:
                a = act[s.ff.fp]
                s.g_gu(h)
                gated_act_planes(s.g_gu.planes, s.g_gu.splits, B, s.ff.fp, s.ff.act, a)
                s.g_down(a)
                y = SublayerOutput(planes=s.g_down.planes)
            last = k + 1 == len(self.subs)
            residual_update(x, y, s.norm, cfg.eps, h, B, W, self.final_norm if last else None, store=not last)
        self._g_head(h)
        g = self._g_head
        _lib.call("ft_splitk_reduce", g.planes, g.splits, B, self.vocab, g.ldp, g.plane_stride, None, self._logits, self._logits.stride(0), 1, _lib.S())
        return self._logits
