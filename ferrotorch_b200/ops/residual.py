"""One f32 residual per token with the RMS norm on every sublayer's output (``x <- x + norm(f(x))``), and the activation of a dense gated feed-forward, on the
fused kernels of ``csrc/kernels/residual_ops.cu``.

Between two projections there is one kernel: it sums the sublayer's partial results, norms them, adds them to the residual and leaves the next projection's
operand (the residual itself, or its norm ahead of the output projection).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _lib
from .moe import interleave_gate_up, linear_rows
from .streams import SublayerOutput, round_up

GATED_ACTS = {"gelu_tanh": 0, "silu": 1}


def residual_embed(ids: torch.Tensor, table: torch.Tensor, scale: float, x: torch.Tensor, h: torch.Tensor, rows: int) -> None:
    """``x = scale * table[ids]`` (f32) and ``h`` the same in the operand type."""
    _lib.call("ft_residual_embed", ids, table, table.stride(0), table.shape[0], scale, x, x.stride(0), h, h.stride(0), int(h.dtype == torch.float32), rows, table.shape[1],
              _lib.S())


def residual_update(x: torch.Tensor, y: SublayerOutput, w: torch.Tensor, eps: float, h: torch.Tensor, rows: int, width: int, last: Optional[torch.Tensor] = None,
                    store: bool = True) -> None:
    """``x += norm(y) * w``; ``h = x``, or ``norm(x) * last`` when the weights of the model's last norm are given. ``w`` and ``last``: f32, padded."""
    p = y.planes
    n = y.count if y.count is not None else p.shape[0]
    _lib.call("ft_residual_update", x, x.stride(0), p, n, p.stride(0), p.stride(1), w, last, eps, h, h.stride(0), int(h.dtype == torch.float32), rows, width, int(store), _lib.S())


@dataclass
class DenseGatedWeights:
    """``down(act(gate x) * up x)``: ``gu`` ``[2 * fp, width]`` (gate and up rows interleaved in eights), ``down`` ``[width, ff]``, both with padded pitches."""
    gu: torch.Tensor
    down: torch.Tensor
    act: str = "gelu_tanh"

    @property
    def fp(self) -> int:
        return self.gu.shape[0] // 2

    @staticmethod
    def pack(gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, device, dtype, act: str = "gelu_tanh") -> "DenseGatedWeights":
        f, width = gate.shape
        gu = interleave_gate_up(gate.to(device, dtype), up.to(device, dtype), round_up(width, 32))
        d = torch.zeros(width, round_up(f, 32), device=device, dtype=dtype)
        d[:, :f] = down.to(device, dtype)
        return DenseGatedWeights(gu[:, :width], d[:, :f], act)


def gated_act_rows(gu: torch.Tensor, fp: int, act: str) -> torch.Tensor:
    """Activation of interleaved gate / up columns ``[rows, 2 * fp]`` -> ``[rows, fp]``."""
    out = torch.empty(gu.shape[0], fp, device=gu.device, dtype=gu.dtype)
    _lib.call("ft_gated_act", gu, gu.stride(0), gu.shape[0], fp, GATED_ACTS[act], out, out.stride(0), int(gu.dtype == torch.float32), _lib.S())
    return out


def gated_act_planes(planes: torch.Tensor, splits: int, rows: int, fp: int, act: str, out: torch.Tensor) -> torch.Tensor:
    """The same from split-K planes of the projection of a few tokens, to bf16 rows."""
    _lib.call("ft_gated_act_planes", planes, splits, planes.stride(1), planes.stride(0), rows, fp, GATED_ACTS[act], out, out.stride(0), _lib.S())
    return out


def dense_gated_rows(h: torch.Tensor, w: DenseGatedWeights) -> SublayerOutput:
    """Any number of token rows (bf16 or f32)."""
    a = gated_act_rows(linear_rows(h, w.gu), w.fp, w.act)
    y = linear_rows(a[:, : w.down.shape[1]], w.down, out_f32=True)
    return SublayerOutput(planes=y.as_strided((1, y.shape[0], y.shape[1]), (0, y.stride(0), 1)))
