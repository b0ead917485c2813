"""Residual streams ("hyper-connections") and the Dynamic Tanh norm on the fused kernels of ``csrc/kernels/stream_ops.cu``.

A model with ``n`` streams keeps ``n`` f32 copies of the residual per token. Ahead of a sublayer they are summed with the weights ``in``; after it the
sublayer's output is added to every stream with the weights ``out`` while the streams are mixed with an ``n x n`` matrix (indexed from, to). With one
stream and unit weights this is the ordinary residual sum. The kernels work per column, so the mixing, the next sublayer's weighted sum and an
element-wise norm are one pass over the streams.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _lib
from ..errors import InvalidArgument


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


def padded_vector(t: torch.Tensor, device, multiple: int = 8) -> torch.Tensor:
    """f32 copy of a vector, zero padded to a multiple of ``multiple`` elements (the kernels read four columns at a time)."""
    v = torch.zeros(round_up(t.numel(), multiple), device=device, dtype=torch.float32)
    v[: t.numel()] = t.reshape(-1).to(device, torch.float32)
    return v


@dataclass
class DynamicTanhWeights:
    """``tanh(alpha x) * w + b``: one scalar, two vectors, f32 on the device (``w`` and ``b`` padded)."""
    alpha: torch.Tensor
    w: torch.Tensor
    b: torch.Tensor

    @staticmethod
    def from_tensors(alpha: torch.Tensor, w: torch.Tensor, b: torch.Tensor, device) -> "DynamicTanhWeights":
        return DynamicTanhWeights(alpha.reshape(1).to(device, torch.float32), padded_vector(w, device), padded_vector(b, device))


@dataclass
class HyperWeights:
    """Connection weights of one sublayer: ``inp`` and ``out`` ``[streams]``, ``mix`` ``[streams, streams]`` (from, to), f32 on the device."""
    inp: torch.Tensor
    mix: torch.Tensor
    out: torch.Tensor

    @staticmethod
    def from_tensors(inp: torch.Tensor, mix: torch.Tensor, out: torch.Tensor, device) -> "HyperWeights":
        f = [t.to(device, torch.float32).contiguous() for t in (inp, mix, out)]
        if f[1].shape != (f[0].numel(), f[0].numel()) or f[2].numel() != f[0].numel():
            raise InvalidArgument("hyper-connections: in [n], mix [n, n] and out [n] must agree")
        return HyperWeights(*f)


@dataclass
class SublayerOutput:
    """What a sublayer hands to the stream update: f32 ``planes`` ``[count, rows, ld]`` to be summed, and / or ``rows`` of expert output with the
    index ``row_of`` ``[tokens, top]`` of the rows that belong to each token, and / or a ``bias``."""
    planes: Optional[torch.Tensor] = None
    rows: Optional[torch.Tensor] = None
    row_of: Optional[torch.Tensor] = None
    top: int = 0
    count: Optional[int] = None          # planes in use when fewer than allocated
    bias: Optional[torch.Tensor] = None  # f32 vector added to every row


def dynamic_tanh(x: torch.Tensor, weights: DynamicTanhWeights, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Dynamic Tanh of the rows of ``x`` ``[rows, width]`` (bf16 or f32, row pitch a multiple of four)."""
    rows, W = x.shape
    if out is None:
        out = torch.empty(rows, round_up(W, 8), device=x.device, dtype=x.dtype)[:, :W]
    _lib.call("ft_dynamic_tanh", x, x.stride(0), weights.alpha, weights.w, weights.b, out, out.stride(0), int(x.dtype == torch.float32), rows, W, _lib.S())
    return out


def hyper_embed(ids: torch.Tensor, table: torch.Tensor, first: DynamicTanhWeights, streams: torch.Tensor, inp: Optional[torch.Tensor], norm: DynamicTanhWeights,
                h: torch.Tensor, rows: int, width: int) -> None:
    """Sets every stream of ``streams`` ``[rows, n, ld]`` to the normalised embedding of the tokens and ``h`` to the first sublayer's operand."""
    _lib.call("ft_hyper_embed", ids, table, table.stride(0), table.shape[0], first.alpha, first.w, first.b, streams, streams.shape[1], streams.stride(1), inp,
              norm.alpha, norm.w, norm.b, h, h.stride(0), int(h.dtype == torch.float32), rows, width, _lib.S())


def hyper_update(streams: torch.Tensor, weights: HyperWeights, y: SublayerOutput, next_inp: Optional[torch.Tensor], norm: DynamicTanhWeights, h: torch.Tensor,
                 rows: int, width: int, store: bool = True) -> None:
    """Adds a sublayer's output to the streams and writes the next operand: ``h = norm(sum_s next_inp[s] x_s)`` (plain sum when ``None``)."""
    p, r = y.planes, y.rows
    n = 0 if p is None else (y.count if y.count is not None else p.shape[0])
    _lib.call("ft_hyper_update", streams, streams.shape[1], streams.stride(1), weights.mix, weights.out, p, n, 0 if p is None else p.stride(0),
              0 if p is None else p.stride(1), r, y.row_of, y.top if r is not None else 0, 0 if r is None else r.stride(0), next_inp, norm.alpha, norm.w, norm.b,
              h, h.stride(0), int(h.dtype == torch.float32), rows, width, int(store), _lib.S())
