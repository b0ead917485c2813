"""One f32 residual per token, with the RMS norm on every sublayer's output (``x <- x + norm(f(x))``) or ahead of two sublayers side by side
(``x <- x + m (f(norm1(x)) + g(norm2(x)))``), averages over the results of all layers so far, the token shift ahead of a mixer, and the activations of dense feed-forwards, on the
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
from .streams import SublayerOutput, padded_vector, round_up

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


def parallel_embed(ids: torch.Tensor, table: torch.Tensor, w1: torch.Tensor, w2: Optional[torch.Tensor], eps: float, x: torch.Tensor, h1: torch.Tensor,
                   h2: Optional[torch.Tensor], rows: int) -> None:
    """``x = table[ids]`` (f32) and the operands of the first layer's two sublayers: ``h1 = norm(x) * w1``, ``h2 = norm(x) * w2`` (``w2`` ``None``: the first alone)."""
    _lib.call("ft_parallel_embed", ids, table, table.stride(0), table.shape[0], w1, w2, eps, x, x.stride(0), h1, h2, h1.stride(0), int(h1.dtype == torch.float32), rows,
              table.shape[1], _lib.S())


def parallel_update(x: torch.Tensor, mult: float, a: Optional[SublayerOutput], b: Optional[SublayerOutput], w1: torch.Tensor, w2: Optional[torch.Tensor], eps: float,
                    h1: torch.Tensor, h2: Optional[torch.Tensor], rows: int, width: int, store: bool = True) -> None:
    """``x += mult * (a + b)`` for what two sublayers of the same ``x`` returned, then the next operands as in :func:`parallel_embed`. ``a`` has planes alone; ``b`` planes,
    expert rows and a bias."""
    def planes(y):
        p = None if y is None else y.planes
        return (None, 0, 0, 0) if p is None else (p, y.count if y.count is not None else p.shape[0], p.stride(0), p.stride(1))
    r = None if b is None else b.rows
    _lib.call("ft_parallel_update", x, x.stride(0), mult, *planes(a), *planes(b), r, None if r is None else b.row_of, 0 if r is None else b.top, 0 if r is None else r.stride(0),
              None if b is None else b.bias, w1, w2, eps, h1, h2, h1.stride(0), int(h1.dtype == torch.float32), rows, width, int(store), _lib.S())


@dataclass
class TokenShift:
    """Ahead of a mixer every column moves from its normed value towards the previous token's by its share in ``share`` (f32, padded). ``state`` ``[slots, ld]`` f32 keeps the last
    normed row of every sequence."""
    share: torch.Tensor
    state: torch.Tensor


def _operand(h, rstd, shift: Optional[TokenShift], slots, positions) -> tuple:
    """What an update does with the norm of the new residual: shared tail of the launchers' arguments."""
    s = shift is not None
    return (h, 0 if h is None else h.stride(0), rstd, shift.share if s else None, shift.state if s else None, shift.state.stride(0) if s else 0, slots if s else None,
            positions if s else None)


def depth_embed(ids: torch.Tensor, table: torch.Tensor, x: torch.Tensor, results: torch.Tensor, w: Optional[torch.Tensor], eps: float, rows: int, h: Optional[torch.Tensor] = None,
                rstd: Optional[torch.Tensor] = None, shift: Optional[TokenShift] = None, slots=None, positions=None) -> None:
    """``x = results[0] = table[ids]`` (f32). Then either ``rstd`` gets the factor of every row's norm (:func:`token_shift` makes the operand of it), or ``h = norm(x) * w``, with
    ``shift`` (one token per sequence, whose state is in ``slots``) shifted."""
    _lib.call("ft_depth_embed", ids, table, table.stride(0), table.shape[0], x, results, x.stride(0), w, eps, *_operand(h, rstd, shift, slots, positions),
              int(table.dtype == torch.float32), rows, table.shape[1], _lib.S())


def depth_update(x: torch.Tensor, results: torch.Tensor, average: torch.Tensor, y: SublayerOutput, w_out: torch.Tensor, w: Optional[torch.Tensor], eps: float, dtype, rows: int,
                 width: int, h: Optional[torch.Tensor] = None, rstd: Optional[torch.Tensor] = None, shift: Optional[TokenShift] = None, slots=None, positions=None,
                 store: bool = True) -> None:
    """``results[n] = x + norm(y) * w_out`` with ``n = len(average) - 1``, ``x = sum_j average[j] results[j]``, then as in :func:`depth_embed`. ``results`` ``[layers + 1, rows, ld]`` and
    ``x`` are f32 with one pitch, ``y`` has planes or expert rows."""
    p, r = y.planes, y.rows
    n = 0 if p is None else (y.count if y.count is not None else p.shape[0])
    _lib.call("ft_depth_update", x, results, results.stride(0), x.stride(0), average.numel() - 1, average, p, n, 0 if p is None else p.stride(0), 0 if p is None else p.stride(1), r,
              None if r is None else y.row_of, 0 if r is None else y.top, 0 if r is None else r.stride(0), w_out, w, eps, *_operand(h, rstd, shift, slots, positions),
              int(dtype == torch.float32), rows, width, int(store), _lib.S())


def token_shift(x: torch.Tensor, rstd: torch.Tensor, w: torch.Tensor, shift: TokenShift, spans: torch.Tensor, seq_of: torch.Tensor, h: torch.Tensor, rows: int, width: int) -> None:
    """``h = n + (n of the token before - n) * share`` with ``n = x * rstd * w`` for a ragged batch: ``spans`` as in :class:`~ferrotorch_b200.models.serving.MemoryPlan`, ``seq_of``
    the sequence of a row. Reads and replaces the states of its sequences."""
    _lib.call("ft_token_shift", x, x.stride(0), rstd, w, shift.share, spans, seq_of, shift.state, shift.state.stride(0), h, h.stride(0), int(h.dtype == torch.float32), rows, width,
              _lib.S())


@dataclass
class DensePolyWeights:
    """``down(act(up x))`` with ``act(z) = a N(z) + b N(z^2) + c N(z^3) + e``, ``N`` dividing a token's neurons by their root mean square: ``up`` ``[ff, width]``, ``down``
    ``[width, ff]`` with padded pitches, ``coef`` f32 ``[4]``."""
    up: torch.Tensor
    down: torch.Tensor
    coef: torch.Tensor
    eps: float

    @property
    def ff(self) -> int:
        return self.up.shape[0]

    @staticmethod
    def pack(up: torch.Tensor, down: torch.Tensor, coef: torch.Tensor, eps: float, device, dtype) -> "DensePolyWeights":
        def place(t):
            m = torch.zeros(t.shape[0], round_up(t.shape[1], 32), device=device, dtype=dtype)
            m[:, : t.shape[1]] = t.to(device, dtype)
            return m[:, : t.shape[1]]
        return DensePolyWeights(place(up), place(down), coef.reshape(4).to(device, torch.float32), eps)


def poly_norm_rows(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    """The activation of rows ``z`` ``[rows, ff]``."""
    out = torch.empty(z.shape[0], round_up(z.shape[1], 8), device=z.device, dtype=z.dtype)[:, : z.shape[1]]
    _lib.call("ft_poly_norm", z, z.stride(0), coef, eps, z.shape[0], z.shape[1], out, out.stride(0), int(z.dtype == torch.float32), _lib.S())
    return out


def poly_norm_planes(planes: torch.Tensor, splits: int, rows: int, coef: torch.Tensor, eps: float, out: torch.Tensor) -> torch.Tensor:
    """The same from split-K planes of the projection of a few tokens, to bf16 rows ``out`` ``[16, ff]``."""
    _lib.call("ft_poly_norm_planes", planes, splits, planes.stride(1), planes.stride(0), coef, eps, rows, out.shape[1], out, out.stride(0), _lib.S())
    return out


def dense_poly_rows(h: torch.Tensor, w: DensePolyWeights) -> SublayerOutput:
    """Any number of token rows (bf16 or f32)."""
    y = linear_rows(poly_norm_rows(linear_rows(h, w.up), w.coef, w.eps), w.down, out_f32=True)
    return SublayerOutput(planes=y.as_strided((1, y.shape[0], y.shape[1]), (0, y.stride(0), 1)))


@dataclass
class DenseGatedWeights:
    """``down(act(gate x) * up x)``: ``gu`` ``[2 * fp, width]`` (gate and up rows interleaved in eights), ``down`` ``[width, ff]``, both with padded pitches; biases (f32),
    if any: ``gu_bias`` in the order of the rows of ``gu``, ``down_bias`` (added by the residual update)."""
    gu: torch.Tensor
    down: torch.Tensor
    act: str = "gelu_tanh"
    gu_bias: Optional[torch.Tensor] = None
    down_bias: Optional[torch.Tensor] = None

    @property
    def fp(self) -> int:
        return self.gu.shape[0] // 2

    @staticmethod
    def pack(gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, device, dtype, act: str = "gelu_tanh", gate_bias=None, up_bias=None, down_bias=None) -> "DenseGatedWeights":
        f, width = gate.shape
        gu = interleave_gate_up(gate.to(device, dtype), up.to(device, dtype), round_up(width, 32))
        d = torch.zeros(width, round_up(f, 32), device=device, dtype=dtype)
        d[:, :f] = down.to(device, dtype)
        gb = db = None
        if gate_bias is not None:
            gb = interleave_gate_up(*(t.reshape(-1, 1).to(device, torch.float32) for t in (gate_bias, up_bias)), 1).flatten().contiguous()
            db = padded_vector(down_bias, device)
        return DenseGatedWeights(gu[:, :width], d[:, :f], act, gb, db)


def gated_act_rows(gu: torch.Tensor, fp: int, act: str, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Activation of interleaved gate / up columns ``[rows, 2 * fp]`` -> ``[rows, fp]``; ``bias`` in the order of the columns."""
    out = torch.empty(gu.shape[0], fp, device=gu.device, dtype=gu.dtype)
    _lib.call("ft_gated_act", gu, gu.stride(0), bias, gu.shape[0], fp, GATED_ACTS[act], out, out.stride(0), int(gu.dtype == torch.float32), _lib.S())
    return out


def gated_act_planes(planes: torch.Tensor, splits: int, rows: int, fp: int, act: str, out: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The same from split-K planes of the projection of a few tokens, to bf16 rows."""
    _lib.call("ft_gated_act_planes", planes, splits, planes.stride(1), planes.stride(0), bias, rows, fp, GATED_ACTS[act], out, out.stride(0), _lib.S())
    return out


def dense_gated_rows(h: torch.Tensor, w: DenseGatedWeights) -> SublayerOutput:
    """Any number of token rows (bf16 or f32)."""
    a = gated_act_rows(linear_rows(h, w.gu), w.fp, w.act, w.gu_bias)
    y = linear_rows(a[:, : w.down.shape[1]], w.down, out_f32=True)
    return SublayerOutput(planes=y.as_strided((1, y.shape[0], y.shape[1]), (0, y.stride(0), 1)), bias=w.down_bias)
