"""Matrix memory (the mLSTM cell of xLSTM) on the kernels of ``csrc/kernels/matrix_memory.cu``: per head an f32 matrix and vector that decay and take in outer products
under log-domain gates with a soft limit, a normalised read-out, a norm per head, an output gate and a scale.

Prompts walk chunks of 128 tokens on the tensor cores, long ones in several segments at the same time; a decode step reads and writes the state once. f32 data and
sizes beyond the walk kernel go token by token.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _lib
from .gqa_attention import pack_head_vector
from .streams import padded_vector, round_up

VALUE_SLICE = 128                    # value columns per CTA of the walk kernel
MAX_DECODE_SIZE = 1024


@dataclass(frozen=True)
class MemoryDims:
    """Sizes of one matrix memory. Projection rows: ``heads x d16`` queries, keys, ``heads x v16`` values, output gates; gate rows: ``h8`` input gates, ``h8``
    forget gates (heads padded to a multiple of 8)."""
    heads: int
    dim: int
    vdim: int
    cap: float
    eps: float
    out_scale: float = 1.0

    @property
    def d16(self): return round_up(self.dim, 16)
    @property
    def v16(self): return round_up(self.vdim, 16)
    @property
    def h8(self): return round_up(self.heads, 8)
    @property
    def gate_col(self): return self.heads * (2 * self.d16 + self.v16)
    @property
    def proj_cols(self): return self.gate_col + self.heads * self.v16
    @property
    def out_cols(self): return self.heads * self.v16
    @property
    def state_size(self):
        """f32 values of a sequence's state: per head the matrix, the normaliser, the running maximum (and three spare)."""
        return self.heads * (self.d16 * self.v16 + self.d16 + 4)

    def walk_supported(self) -> bool:
        return bool(_lib.kernels().ft_mm_walk_fits(self.dim, self.vdim))

    def decode_supported(self) -> bool:
        return max(self.d16, self.v16) <= MAX_DECODE_SIZE


@dataclass
class MemoryWeights:
    """Vectors of a matrix memory (f32 on the device): biases of the input and forget gates, weight of the output norm."""
    dims: MemoryDims
    bias_i: torch.Tensor
    bias_f: torch.Tensor
    norm: torch.Tensor

    @staticmethod
    def pack(dims: MemoryDims, bias_i, bias_f, norm, device) -> "MemoryWeights":
        return MemoryWeights(dims, padded_vector(bias_i, device), padded_vector(bias_f, device), pack_head_vector(norm, dims.heads, dims.vdim, device))


def matrix_memory_rows(x: torch.Tensor, gates: torch.Tensor, w: MemoryWeights, batch, states: torch.Tensor, out: torch.Tensor, walk: Optional[bool] = None) -> torch.Tensor:
    """New tokens of a ragged batch into ``out`` ``[rows, out_cols]``; ``x``: projection rows, ``gates``: f32 gate pre-activations, ``states`` ``[slots, state_size]`` is
    advanced. ``walk=False`` forces the token-by-token kernel."""
    D, T, S = w.dims, x.shape[0], _lib.S()
    f32 = x.dtype == torch.float32
    walk = not f32 and D.walk_supported() if walk is None else walk
    plan = batch.memory_plan(D.heads * -(-D.v16 // VALUE_SLICE) if walk else 0)
    o = torch.empty(T, D.out_cols, device=x.device, dtype=x.dtype)
    nm = torch.empty(plan.sequences, D.heads * (D.d16 + 4), device=x.device, dtype=torch.float32)
    vectors = (gates, gates.stride(0), w.bias_i, w.bias_f, D.cap)
    head = (x, x.stride(0), T, *vectors)
    if walk:
        scratch = torch.empty(plan.scratch * D.state_size, device=x.device, dtype=torch.float32) if plan.scratch else None
        if plan.scratch:
            _lib.call("ft_mm_walk", *head, plan.inner, plan.inner.shape[0], D.heads, D.dim, D.vdim, states, states.stride(0), scratch, None, None, 0, S)
            _lib.call("ft_mm_merge", plan.chains, plan.sequences, D.heads, D.dim, D.vdim, states, states.stride(0), scratch, S)
        _lib.call("ft_mm_walk", *head, plan.segments, plan.segments.shape[0], D.heads, D.dim, D.vdim, states, states.stride(0), scratch, nm, o, 1, S)
    else:
        _lib.call("ft_mm_rows", x, x.stride(0), *vectors, plan.segments, plan.segments.shape[0], D.heads, D.dim, D.vdim, states, states.stride(0), nm, o, int(f32), S)
    gate = x[:, D.gate_col:]
    _lib.call("ft_mm_finish", o, T, gate, gate.stride(0), w.norm, D.eps, D.out_scale, out, out.stride(0), D.heads, D.dim, D.vdim, plan.chains, plan.sequences, nm, states,
              states.stride(0), int(f32), S)
    return out


def matrix_memory_decode(planes: torch.Tensor, splits: int, w: MemoryWeights, state, states: torch.Tensor, B: int, col: int, gate_col: int, out: torch.Tensor) -> None:
    """One token per sequence from split-K planes (projection columns from ``col``, gate columns from ``gate_col``) into bf16 rows ``out``; advances ``states``."""
    D = w.dims
    _lib.call("ft_mm_decode", planes, splits, planes.stride(1), planes.stride(0), B, D.heads, D.dim, D.vdim, col, gate_col, w.bias_i, w.bias_f, D.cap, w.norm, D.eps, D.out_scale,
              state.positions, state.slots, states, states.stride(0), out, out.stride(0), _lib.S())
