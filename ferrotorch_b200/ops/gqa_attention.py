"""Grouped-query attention over a paged row cache on the kernels of ``csrc/kernels/gqa_attn.cu``: own key and value sizes, optional RMS norms on queries and keys (per
head or over the whole projection), rotary positions on the first dimensions (neighbouring pairs or halves), an optional sliding window beside which the first tokens
may stay visible, or chunks of the sequence that do not see one another, an optional sink per head, values optionally mixed with an earlier layer's, an output gate (per
element or per head) and a scale. Differential heads subtract the outputs of two maps over the same values and norm the result. A layer may read the keys and values
that an earlier layer cached.

Prompts of any ragged batch run a tcgen05 flash kernel that reads keys and values from the pages (both maps of a differential head in one CTA); a decode step streams the
visible rows once for all heads of a group and both maps. f32 data takes a plain kernel.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _lib
from .streams import padded_vector, round_up

GATE_NONE, GATE_ELEMENT, GATE_HEAD = 0, 1, 2
NORM_HEAD, NORM_WHOLE, NORM_NONE = 0, 1, 2
SMALL_TOKENS = 16
GROUP_ROWS = 128                     # query rows (tokens x heads of a group) of a flash sub-tile
MAX_SPLITS = 64


@dataclass(frozen=True)
class GqaDims:
    """Sizes and constants of one attention layer. ``window`` 0: every earlier position is visible; otherwise the last ``window`` and the first ``keep`` of them are.
    ``chunk`` > 0: only positions of the same chunk of the sequence are. ``halves``: dimension i turns with i + rot_dims / 2 instead of 2 i with 2 i + 1. ``norm``: whether queries
    and keys are normed. ``maps`` 2: differential heads, two queries and keys each, ``diff`` in their norm's factor ``1 - diff``. ``own`` False: keys and values are an earlier
    layer's. Head sizes are padded to multiples of 16: projection rows ``heads x maps x d16 | kv_heads x maps x d16 | kv_heads x v16`` (queries alone without ``own``), cache rows
    ``kv_heads x maps x d16 | kv_heads x v16``."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_dims: int
    scale: float
    eps: float
    window: int = 0
    whole_norm: bool = False
    gate: int = GATE_NONE
    out_scale: float = 1.0
    keep: int = 0
    halves: bool = False
    norm: bool = True
    chunk: int = 0
    maps: int = 1
    diff: float = 0.0
    own: bool = True

    @property
    def norm_kind(self): return (NORM_WHOLE if self.whole_norm else NORM_HEAD) if self.norm else NORM_NONE
    @property
    def d16(self): return round_up(self.dim, 16)
    @property
    def v16(self): return round_up(self.vdim, 16)
    @property
    def k_col(self): return self.heads * self.maps * self.d16
    @property
    def v_col(self): return self.k_col + self.kv_heads * self.maps * self.d16
    @property
    def qkv_cols(self): return self.v_col + self.kv_heads * self.v16 if self.own else self.k_col
    @property
    def out_cols(self): return self.heads * self.v16
    @property
    def row(self): return self.kv_heads * (self.maps * self.d16 + self.v16)
    @property
    def turned(self): return self.norm or self.rot_dims > 0          # whether queries are changed ahead of the scores

    def flash_tile(self) -> int:
        """Tokens per tile of the flash kernel, 0 when these sizes do not fit it."""
        return _lib.kernels().ft_gqa_flash_subtiles(self.heads, self.kv_heads, self.dim, self.vdim, self.maps) * (GROUP_ROWS // (self.heads // self.kv_heads))

    def decode_supported(self) -> bool:
        return bool(_lib.kernels().ft_gqa_decode_fits(self.heads, self.kv_heads, self.dim, self.vdim, self.maps))


def pack_head_rows(w: torch.Tensor, heads: int, size: int, device, dtype) -> torch.Tensor:
    """``[heads * size, k]`` -> ``[heads * padded size, k]`` with zero rows behind every head."""
    out = torch.zeros(heads, round_up(size, 16), w.shape[1], device=device, dtype=dtype)
    out[:, :size] = w.to(device, dtype).reshape(heads, size, -1)
    return out.flatten(0, 1)


def pack_head_columns(w: torch.Tensor, heads: int, size: int, device, dtype) -> torch.Tensor:
    """``[n, heads * size]`` -> ``[n, heads * padded size]``."""
    out = torch.zeros(w.shape[0], heads, round_up(size, 16), device=device, dtype=dtype)
    out[:, :, :size] = w.to(device, dtype).reshape(-1, heads, size)
    return out.flatten(1)


def pack_head_vector(v: torch.Tensor, heads: int, size: int, device) -> torch.Tensor:
    """f32 vector ``[heads * size]`` in the padding of the heads."""
    return pack_head_columns(v.reshape(1, -1), heads, size, device, torch.float32)[0].contiguous()


@dataclass
class GqaWeights:
    """Vectors of an attention layer (f32 on the device): query and key norm weights, ``sink`` ``[heads]``, ``mix`` (the weight of an earlier layer's values). ``blend``: the
    factor of a differential head's second map."""
    dims: GqaDims
    q_norm: Optional[torch.Tensor]
    k_norm: Optional[torch.Tensor]
    sink: Optional[torch.Tensor] = None
    mix: Optional[torch.Tensor] = None
    blend: float = 0.0

    @staticmethod
    def pack(dims: GqaDims, q_norm, k_norm, device, sink=None, mix=None, blend: float = 0.0) -> "GqaWeights":
        hq, hk = (dims.heads, dims.kv_heads) if dims.whole_norm else (1, 1)
        qw, kw = (pack_head_vector(t, n, dims.dim, device) if dims.norm else None for t, n in ((q_norm, hq), (k_norm, hk)))
        return GqaWeights(dims, qw, kw,
                          None if sink is None else padded_vector(sink, device), None if mix is None else mix.reshape(1).to(device, torch.float32), blend)


def differential_blend(lq1: torch.Tensor, lk1: torch.Tensor, lq2: torch.Tensor, lk2: torch.Tensor, diff: float) -> float:
    """The factor of the second map: ``exp(lq1 . lk1) - exp(lq2 . lk2) + diff``."""
    a, b = ((q.double() * k.double()).sum().exp() for q, k in ((lq1, lk1), (lq2, lk2)))
    return float(a - b) + diff


def gqa_attention_rows(qkv: torch.Tensor, w: GqaWeights, batch, cache: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, gate: Optional[torch.Tensor], out: torch.Tensor,
                       first_values: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention of a ragged batch of new tokens into ``out`` ``[rows, out_cols]``. ``qkv``: projection rows (their queries are normed and turned in place);
    ``gate``: pre-activations ``[rows, out_cols]`` in the data type or ``[rows, heads]`` f32; ``first_values`` ``[rows, kv_heads * v16]``: mixed in with
    ``w.mix``. ``batch`` holds the tables of :class:`~ferrotorch_b200.models.serving.RowBatch`, ``cache`` is this layer's page storage."""
    D, T, S = w.dims, qkv.shape[0], _lib.S()
    f32 = qkv.dtype == torch.float32
    if D.own or D.turned:
        _lib.call("ft_gqa_prep", qkv, qkv.stride(0), T, D.heads, D.kv_heads, D.dim, D.vdim, D.maps, D.rot_dims, D.norm_kind, int(D.halves), w.q_norm, w.k_norm, D.eps, batch.positions,
                  cos, sin, batch.slots, cache if D.own else None, first_values, 0 if first_values is None else first_values.stride(0), None if first_values is None else w.mix,
                  int(f32), S)
    bt = batch.block_table
    sizes = (D.heads, D.kv_heads, D.dim, D.vdim, D.maps, D.scale, D.window, D.keep, D.chunk, w.sink, gate, 0 if gate is None else gate.stride(0), D.gate, D.out_scale)
    tile = 0 if f32 else D.flash_tile()
    joined = D.maps == 1 or (tile and _lib.kernels().ft_gqa_flash_joins_maps(D.dim, D.vdim))
    to = out if joined else torch.empty(T, D.heads * D.maps * D.v16, device=qkv.device, dtype=torch.float32)
    if tile:
        tiles = batch.query_tiles(tile)
        _lib.call("ft_gqa_flash", qkv, qkv.stride(0), T, cache, cache.shape[0], bt, bt.shape[1], tiles, tiles.shape[0], *sizes, w.blend, 1.0 - D.diff, D.eps, to, to.stride(0),
                  int(not joined), S)
    else:
        _lib.call("ft_gqa_rows", qkv, qkv.stride(0), cache, bt, bt.shape[1], batch.seq_of, batch.positions, T, *sizes, to, to.stride(0), int(not joined), int(f32), S)
    if not joined:
        _lib.call("ft_gqa_differential", to, to.stride(0), T, D.heads, D.vdim, w.blend, 1.0 - D.diff, D.eps, out, out.stride(0), int(f32), S)
    return out


class GqaDecodeBuffers:
    """Scratch of the decode kernels for one layer size (shared by layers of the same size, which run one after another)."""

    def __init__(self, dims: GqaDims, max_batch: int, max_tokens: int, device, splits: Optional[int] = None):
        D = dims
        groups = D.kv_heads * -(-(D.heads * D.maps // D.kv_heads) // 16)
        span = min(max_tokens, D.window + D.keep if D.window else max_tokens, D.chunk or max_tokens)
        # by batch size: two CTAs per SM, at least one 64-row chunk per split at the longest visible range
        self.splits = [splits or max(1, min(MAX_SPLITS, 296 // (b * groups), -(-span // 64))) for b in range(1, max_batch + 1)]
        self.q = torch.zeros(SMALL_TOKENS, D.heads * D.maps, D.maps * D.d16, device=device, dtype=torch.bfloat16)      # a map's query stays zero outside its own part
        self.gate = torch.zeros(SMALL_TOKENS, D.out_cols if D.gate == GATE_ELEMENT else D.heads, device=device)
        self.ws = torch.zeros(max(b * n for b, n in enumerate(self.splits, 1)) * groups * 16 * (D.v16 + 4), device=device)
        self.counters = torch.zeros(SMALL_TOKENS * groups, device=device, dtype=torch.int32)


def gqa_attention_decode(planes: torch.Tensor, splits: int, w: GqaWeights, b: GqaDecodeBuffers, state, cache: torch.Tensor, cos, sin, B: int, gate_col: int, out: torch.Tensor,
                         keep_values: Optional[torch.Tensor] = None, first_values: Optional[torch.Tensor] = None) -> None:
    """One token per sequence from the split-K planes of the projection (columns ``qkv_cols`` from 0 on, the gate's pre-activations at ``gate_col``) into ``out``
    ``[16, out_cols]``. ``keep_values`` (f32 ``[16, kv_heads * v16]``) receives the values, ``first_values`` such values are mixed in."""
    D, S = w.dims, _lib.S()
    bt, mb = state.block_table, state.block_table.shape[1]
    _lib.call("ft_gqa_decode_prep", planes, splits, planes.stride(1), planes.stride(0), B, D.heads, D.kv_heads, D.dim, D.vdim, D.maps, D.rot_dims, D.norm_kind, int(D.halves),
              w.q_norm, w.k_norm, D.eps, state.positions, cos, sin, bt, mb, gate_col, D.gate, b.gate, keep_values, first_values, None if first_values is None else w.mix, b.q,
              cache if D.own else None, S)
    _lib.call("ft_gqa_decode", b.q, cache, bt, mb, state.seq_lens, B, D.heads, D.kv_heads, D.dim, D.vdim, D.maps, D.scale, D.window, D.keep, D.chunk, w.sink, b.gate, D.gate,
              D.out_scale, w.blend, 1.0 - D.diff, D.eps, b.splits[B - 1], b.ws, b.counters, out, out.stride(0), S)
