"""Selective state space (the recurrence of Mamba-2) on the kernels of ``csrc/kernels/state_space.cu``: a short causal convolution, per head an f32 matrix that decays and takes in
outer products with a step size per token, a skip connection, a gate, and an RMS norm over equal parts of the output.

Prompts walk chunks of 128 tokens on the tensor cores, long ones in several segments at the same time; a decode step reads and writes the state once. f32 data and sizes beyond
the walk kernel go token by token.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _lib
from ..errors import InvalidArgument
from .gqa_attention import pack_head_columns, pack_head_rows, pack_head_vector
from .streams import padded_vector, round_up

SMALL_TOKENS = 16
VALUE_SLICE = 64                     # value columns per CTA of the walk kernel, of which two share an SM
MAX_COLUMNS = 16384                  # heads x padded value size that the norm takes
MAX_PARTS, MAX_DECODE_STATE = 4096, 4096


@dataclass(frozen=True)
class SsmDims:
    """Sizes of one state-space mixer: ``state`` (N) is shared within ``groups`` of heads; ``taps`` of the convolution; ``parts`` of the norm. Projection rows in the kernels'
    padding: gate ``heads x v16`` | values ``heads x v16`` | B ``groups x n16`` | C ``groups x n16``, then ``h8`` step sizes (heads padded to a multiple of 8)."""
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    parts: int
    eps: float

    @property
    def v16(self): return round_up(self.vdim, 16)
    @property
    def n16(self): return round_up(self.state, 16)
    @property
    def h8(self): return round_up(self.heads, 8)
    @property
    def out_cols(self): return self.heads * self.v16
    @property
    def channels(self): return self.out_cols + 2 * self.groups * self.n16
    @property
    def main(self):
        """Columns ahead of the step sizes."""
        return self.out_cols + self.channels
    @property
    def state_size(self):
        """f32 values of a sequence's state: the matrices, then the last inputs of the convolution."""
        return self.heads * self.n16 * self.v16 + (self.taps - 1) * self.channels

    def validate(self) -> None:
        if min(self.heads, self.vdim, self.state, self.groups, self.taps, self.parts) < 1 or self.heads % self.groups or (self.heads * self.vdim) % self.parts:
            raise InvalidArgument("state space: sizes must be positive, heads a multiple of groups and heads x vdim of the norm's parts")
        if self.out_cols > MAX_COLUMNS or self.parts > MAX_PARTS:
            raise InvalidArgument(f"state space: at most {MAX_COLUMNS} output columns and {MAX_PARTS} parts of the norm")

    def walk_supported(self) -> bool:
        return bool(_lib.kernels().ft_ssm_walk_fits(self.state))

    def decode_supported(self) -> bool:
        return self.n16 <= MAX_DECODE_STATE


@dataclass
class SsmWeights:
    """Vectors of a state-space mixer (f32 on the device): ``conv`` ``[taps, channels]`` (the current token's weight last), its bias, bias of the step sizes, ``rate`` (-e^A_log),
    ``skip`` (D), weight of the norm."""
    dims: SsmDims
    conv: torch.Tensor
    conv_bias: torch.Tensor
    dt_bias: torch.Tensor
    rate: torch.Tensor
    skip: torch.Tensor
    norm: torch.Tensor

    @staticmethod
    def _channels(dims: SsmDims, t: torch.Tensor, device, dtype, pack) -> list:
        """Rows ``[values | B | C]`` of the checkpoint in the kernels' padding."""
        D = dims
        parts = torch.split(t, [D.heads * D.vdim, D.groups * D.state, D.groups * D.state])
        return [pack(p, n, s, device, dtype) for p, n, s in zip(parts, (D.heads, D.groups, D.groups), (D.vdim, D.state, D.state))]

    @staticmethod
    def pack(dims: SsmDims, conv, conv_bias, dt_bias, a_log, skip, norm, device) -> "SsmWeights":
        D, f32 = dims, torch.float32
        w = torch.cat(SsmWeights._channels(D, conv, device, f32, pack_head_rows)).t().contiguous()
        b = torch.cat(SsmWeights._channels(D, conv_bias.reshape(-1, 1), device, f32, pack_head_rows)).flatten().contiguous()
        return SsmWeights(D, w, b, padded_vector(dt_bias, device), padded_vector(-torch.exp(a_log.to(device, f32)), device), padded_vector(skip, device),
                          pack_head_vector(norm, D.heads, D.vdim, device))

    @staticmethod
    def pack_projection(dims: SsmDims, w, device, dtype) -> torch.Tensor:
        """``[gate | values | B | C | step sizes]`` rows of the checkpoint -> ``[main + h8, width]``."""
        D = dims
        inner = D.heads * D.vdim
        z, xbc, dt = torch.split(w, [inner, inner + 2 * D.groups * D.state, D.heads])
        steps = torch.zeros(D.h8, w.shape[1], device=device, dtype=dtype)
        steps[: D.heads] = dt.to(device, dtype)
        return torch.cat([pack_head_rows(z, D.heads, D.vdim, device, dtype), *SsmWeights._channels(D, xbc, device, dtype, pack_head_rows), steps])

    @staticmethod
    def pack_output(dims: SsmDims, w, device, dtype) -> torch.Tensor:
        return pack_head_columns(w, dims.heads, dims.vdim, device, dtype)


def state_space_rows(x: torch.Tensor, dt: torch.Tensor, w: SsmWeights, batch, states: torch.Tensor, walk: Optional[bool] = None) -> torch.Tensor:
    """New tokens of a ragged batch: returns ``[rows, out_cols]``, normed. ``x``: projection rows (``main`` columns), ``dt``: f32 step sizes ahead of bias and softplus, ``states``
    ``[slots, state_size]`` is advanced. ``walk=False`` forces the token-by-token kernel."""
    D, T, S = w.dims, x.shape[0], _lib.S()
    f32 = x.dtype == torch.float32
    walk = not f32 and D.walk_supported() if walk is None else walk
    plan = batch.memory_plan(-(-D.heads * -(-D.v16 // VALUE_SLICE) // 2) if walk else 0)
    sizes, stride = (D.heads, D.groups, D.state, D.vdim), states.stride(0)
    xbc = x[:, D.out_cols: D.main]
    u = torch.empty(T, D.channels, device=x.device, dtype=x.dtype)
    _lib.call("ft_ssm_conv", xbc, x.stride(0), T, batch.seq_of, plan.spans, w.conv, w.conv_bias, states, stride, *sizes, D.taps, u, int(f32), S)
    y = torch.empty(T, D.out_cols, device=x.device, dtype=x.dtype)
    vectors = (dt, dt.stride(0), w.dt_bias, w.rate, w.skip)
    if walk:
        scratch = torch.empty(plan.scratch * D.heads * (D.n16 * D.v16 + 4), device=x.device, dtype=torch.float32) if plan.scratch else None
        if plan.scratch:
            _lib.call("ft_ssm_walk", u, T, *vectors, plan.inner, plan.inner.shape[0], *sizes, states, stride, scratch, None, 0, S)
            _lib.call("ft_ssm_merge", plan.chains, plan.sequences, *sizes, states, stride, scratch, S)
        _lib.call("ft_ssm_walk", u, T, *vectors, plan.segments, plan.segments.shape[0], *sizes, states, stride, scratch, y, 1, S)
    else:
        _lib.call("ft_ssm_rows", u, *vectors, plan.segments, plan.segments.shape[0], *sizes, states, stride, y, int(f32), S)
    out = torch.empty(T, D.out_cols, device=x.device, dtype=x.dtype)
    _lib.call("ft_ssm_finish", y, T, x, x.stride(0), D.parts, D.eps, w.norm, out, out.stride(0), *sizes, D.taps, xbc, x.stride(0), plan.spans, plan.sequences, states, stride,
              int(f32), S)
    return out


class SsmDecodeBuffers:
    """Scratch of the decode kernels for one layer size (shared by layers of the same size, which run one after another)."""

    def __init__(self, dims: SsmDims, device):
        D = dims
        self.u = torch.zeros(SMALL_TOKENS, D.channels, device=device)
        self.gz, self.gated = torch.zeros(2, SMALL_TOKENS, D.out_cols, device=device)
        self.step = torch.zeros(SMALL_TOKENS, 2 * D.heads, device=device)
        self.counters = torch.zeros(SMALL_TOKENS, device=device, dtype=torch.int32)
        self.out = torch.zeros(SMALL_TOKENS, D.out_cols, device=device, dtype=torch.bfloat16)


def state_space_decode(planes: torch.Tensor, splits: int, w: SsmWeights, b: SsmDecodeBuffers, state, states: torch.Tensor, B: int) -> torch.Tensor:
    """One token per sequence from split-K planes of the projection (``main`` columns, then the step sizes): returns normed bf16 rows ``[16, out_cols]`` (in ``b``); advances
    ``states``."""
    D = w.dims
    _lib.call("ft_ssm_decode", planes, splits, planes.stride(1), planes.stride(0), B, D.heads, D.groups, D.state, D.vdim, D.taps, 0, D.out_cols, D.main, w.conv, w.conv_bias, w.dt_bias,
              w.rate, w.skip, D.parts, D.eps, w.norm, state.positions, state.slots, states, states.stride(0), b.u, b.gz, b.step, b.gated, b.counters, b.out, b.out.stride(0), _lib.S())
    return b.out
