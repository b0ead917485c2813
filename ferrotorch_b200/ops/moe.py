"""Mixture of experts on the kernels of ``csrc/kernels/moe.cu``: sigmoid or softmax router, the ``top`` best experts per token, experts of the clamped gated form
``W_down (g sigmoid(slope g) (u + 1))`` with ``g = min(W_gate x, limit)`` and ``u = clamp(W_up x, -limit, limit)`` applied to ``score * x``, or of the form
``score * W_down (silu(W_gate x) * (W_up x))``, and an optional expert that every token passes through. The choice goes by logit or by a :class:`RouteRule`.

Prompts sort their (token, expert) pairs into 128-row segments and run grouped tcgen05 GEMMs; a decode step (up to 16 tokens in bf16) streams the
weights of the experts in use through ``mma.sync`` with all tokens in shared memory.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence

import torch

from .. import _lib
from ..errors import InvalidArgument
from .gemm import gemm
from .streams import SublayerOutput, round_up

SMALL_TOKENS = 16
MAX_TOP = 32
_SMALL_SMEM = 208 * 1024
SEGMENT = 128


def linear_rows(x: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None, out_f32: bool = False) -> torch.Tensor:
    """``x @ w.T`` for row-major matrices with padded pitches: tcgen05 GEMM for bf16, exact FMA-pipe GEMM for f32. Returns ``[rows, N]``, a view of a
    buffer whose rows start on 16-byte boundaries."""
    M, N, K = x.shape[0], w.shape[0], w.shape[1]
    f32 = x.dtype == torch.float32
    if out is None:
        out = torch.empty(M, round_up(N, 8), device=x.device, dtype=torch.float32 if (f32 or out_f32) else x.dtype)[:, :N]
    if not f32:
        return gemm(x, w, out=out)
    _lib.call("ft_gemm_simt", 0, x, w, out, 1, M, N, K, x.stride(0), w.stride(0), out.stride(0), 0, 0, 0, 0, 1, 1.0, 0.0, _lib.S())
    return out


def grouped_linear(x: torch.Tensor, w: torch.Tensor, tile_group: torch.Tensor, n: int, k: int, out: torch.Tensor) -> torch.Tensor:
    """``out[r, :n] = x[r, :k] @ w[g, :n, :k].T`` with ``g = tile_group[r // 128]`` (rows of tiles marked -1 are left alone)."""
    if x.dtype == torch.float32:
        _lib.call("ft_gemm_simt_grouped", x, w, out, x.shape[0], n, k, x.stride(0), w.stride(1), out.stride(0), tile_group, w.stride(0), _lib.S())
    else:
        _lib.call("ft_gemm_grouped", x, w, out, x.shape[0], n, k, x.stride(0), w.stride(1), out.stride(0), int(out.dtype == torch.float32), tile_group, w.shape[0],
                  w.shape[1], _lib.S())
    return out


def interleave_gate_up(gate: torch.Tensor, up: torch.Tensor, ld: int) -> torch.Tensor:
    """``[2 * fp, ld]``: blocks of eight gate rows followed by the eight up rows of the same neurons, zero padded (``fp`` = neurons rounded up to 8)."""
    f, k = gate.shape
    fp = round_up(f, 8)
    w = torch.zeros(fp // 8, 2, 8, ld, device=gate.device, dtype=gate.dtype)
    for i, t in enumerate((gate, up)):
        full = torch.zeros(fp, ld, device=gate.device, dtype=gate.dtype)
        full[:f, :k] = t
        w[:, i] = full.view(fp // 8, 8, ld)
    return w.view(2 * fp, ld)


@dataclass
class ExpertStack:
    """Packed weights of experts of one size: ``gu`` ``[experts, 2 * fp, ld_in]`` (interleaved), ``down`` ``[experts, rows, ld_mid]``."""
    gu: torch.Tensor
    down: torch.Tensor
    ff: int
    limit: float

    @property
    def fp(self) -> int:
        return round_up(self.ff, 8)

    @staticmethod
    def pack(gates: Sequence[torch.Tensor], ups: Sequence[torch.Tensor], downs: Sequence[torch.Tensor], limit: float, device, dtype) -> "ExpertStack":
        f, width = gates[0].shape
        ld_in, ld_mid, rows = round_up(width, 32), round_up(f, 32), round_up(width, 16)
        n = len(gates)
        gu = torch.zeros(n, 2 * round_up(f, 8), ld_in, device=device, dtype=dtype)
        down = torch.zeros(n, rows, ld_mid, device=device, dtype=dtype)
        for i in range(n):
            gu[i] = interleave_gate_up(gates[i].to(device, dtype), ups[i].to(device, dtype), ld_in)
            down[i, :width, :f] = downs[i].to(device, dtype)
        return ExpertStack(gu, down, f, float(limit))


@dataclass
class RouteRule:
    """Experts are chosen by ``sigmoid(logit) + correction`` (``softmax``: by ``logit + correction``), within the ``keep`` best of ``groups`` equal groups of neighbours (0: no
    groups; a group's score is the sum of its two best), and weighted with the chosen sigmoids divided by their sum (``softmax``: the softmax over the chosen sums), times
    ``scale``. ``correction``: f32 ``[experts]`` on the device."""
    correction: torch.Tensor
    groups: int = 0
    keep: int = 0
    scale: float = 1.0
    softmax: bool = False


EXPERT_FORMS = {"clamped": 0, "silu": 1}


@dataclass
class MoeWeights:
    router: torch.Tensor                     # [experts, width] view with a pitch that is a multiple of 8
    experts: ExpertStack
    shared: Optional[ExpertStack]
    width: int
    top: int
    slope: float = 1.702
    form: str = "clamped"
    rule: Optional[RouteRule] = None

    @property
    def kind(self) -> int:
        return EXPERT_FORMS[self.form]

    @property
    def rule_args(self) -> tuple:
        r = self.rule
        return (2 if r.softmax else 1, r.correction, r.groups, r.keep, r.scale) if r else (0, None, 0, 0, 1.0)

    @property
    def num_experts(self) -> int:
        return self.router.shape[0]

    def small_supported(self) -> bool:
        """Whether a decode step of these sizes fits the streaming kernels (tokens in shared memory)."""
        k = max(self.width, self.experts.ff, self.shared.ff if self.shared else 0)
        return self.top <= MAX_TOP and 8 * (2 * round_up(k, 32) + 64) + 128 <= _SMALL_SMEM


@dataclass
class MoeSmallBuffers:
    """Scratch of a decode step, allocated once: routing lists, activations, and one f32 output plane per expert slot plus one for the shared expert."""
    logits: torch.Tensor
    counter: torch.Tensor
    n_active: torch.Tensor
    ids: torch.Tensor
    cnt: torch.Tensor
    pair: torch.Tensor
    pair_of: torch.Tensor
    score: torch.Tensor
    act: torch.Tensor
    act_sh: torch.Tensor
    planes: torch.Tensor

    @staticmethod
    def allocate(weights: Sequence[MoeWeights], device) -> "MoeSmallBuffers":
        E, top, width = (max(getattr(w, k) for w in weights) for k in ("num_experts", "top", "width"))
        f = max(w.experts.ff for w in weights)
        fs = max((w.shared.ff if w.shared else 8) for w in weights)

        def ints(*s):
            return torch.zeros(*s, device=device, dtype=torch.int32)
        return MoeSmallBuffers(torch.zeros(2 * SMALL_TOKENS * E, device=device), ints(1), ints(1), ints(E), ints(E), ints(E * SMALL_TOKENS), ints(E * SMALL_TOKENS),
                               torch.zeros(SMALL_TOKENS * top, device=device), torch.zeros(SMALL_TOKENS * top, round_up(f, 8), device=device, dtype=torch.bfloat16),
                               torch.zeros(SMALL_TOKENS, round_up(fs, 8), device=device, dtype=torch.bfloat16),
                               torch.zeros(top + 1, SMALL_TOKENS, round_up(width, 8), device=device))


def moe_small(h: torch.Tensor, w: MoeWeights, b: MoeSmallBuffers, tokens: int) -> SublayerOutput:
    """Decode step: ``tokens`` (<= 16) bf16 rows of ``h``. The result's planes live in ``b`` until the next call."""
    E, x, s, S = w.num_experts, w.experts, w.shared, _lib.S()
    route = (b.n_active, b.ids, b.cnt, b.pair, b.pair_of, b.score)
    _lib.call("ft_moe_route_small", h, h.stride(0), w.router, w.router.stride(0), tokens, w.width, E, w.top, *w.rule_args, b.logits, b.counter,
              *route, S)
    _lib.call("ft_moe_gate_up_small", h, h.stride(0), tokens, w.width, E, w.top, *route, x.gu, x.ff, x.gu.stride(1), x.limit, s.gu if s else None, s.ff if s else 0,
              s.gu.stride(1) if s else 0, s.limit if s else 0.0, w.kind, w.slope, b.act, b.act.stride(0), b.act_sh, b.act_sh.stride(0), S)
    _lib.call("ft_moe_down_small", b.act, b.act.stride(0), b.act_sh, b.act_sh.stride(0), tokens, w.width, E, w.top, *route, x.down, x.ff, x.down.stride(1),
              s.down if s else None, s.ff if s else 0, s.down.stride(1) if s else 0, x.down.shape[1], b.planes, b.planes.stride(0), b.planes.stride(1), S)
    return SublayerOutput(planes=b.planes, count=w.top + (1 if s else 0))


def gated_act(gu: torch.Tensor, fp: int, limit: float, slope: float, row_score: Optional[torch.Tensor] = None, rows_used: Optional[torch.Tensor] = None,
              form: str = "clamped") -> torch.Tensor:
    """Activation of interleaved gate / up columns ``[rows, 2 * fp]`` -> ``[rows, fp]``; clamped: both scaled by ``row_score`` first, silu: the result is."""
    act = torch.empty(gu.shape[0], fp, device=gu.device, dtype=gu.dtype)
    _lib.call("ft_moe_act", gu, gu.stride(0), row_score, rows_used, gu.shape[0], fp, EXPERT_FORMS[form], limit, slope, act, act.stride(0), int(gu.dtype == torch.float32), _lib.S())
    return act


@dataclass
class MoeRouting:
    """Where every (token, slot) pair of a batch goes: ``expert`` and ``score`` ``[tokens, top]``, ``row_of`` (row in the sorted matrix), tile table."""
    expert: torch.Tensor
    score: torch.Tensor
    pos: torch.Tensor
    start: torch.Tensor
    tile_group: torch.Tensor
    rows_used: torch.Tensor

    @staticmethod
    def choose(h: torch.Tensor, w: MoeWeights) -> "MoeRouting":
        T, E, dev = h.shape[0], w.num_experts, h.device
        logits = linear_rows(h, w.router, out_f32=True)
        tiles = T * w.top // SEGMENT + min(E, T * w.top)
        ints = torch.empty(2 * T * w.top + E + tiles + 1, device=dev, dtype=torch.int32)
        expert, pos, start, group, used = torch.split(ints, [T * w.top, T * w.top, E, tiles, 1])
        score = torch.empty(T * w.top, device=dev, dtype=torch.float32)
        count = torch.zeros(E, device=dev, dtype=torch.int32)
        _lib.call("ft_moe_topk", logits, logits.stride(0), T, E, w.top, *w.rule_args, expert, score, pos, count, _lib.S())
        _lib.call("ft_moe_layout", count, E, tiles, start, group, used, _lib.S())
        return MoeRouting(expert, score, pos, start, group, used)


def moe_rows(h: torch.Tensor, w: MoeWeights) -> SublayerOutput:
    """Any number of token rows ``h`` ``[T, width]`` (bf16 or f32, row pitch a multiple of 8)."""
    T, es, x, s = h.shape[0], h.element_size(), w.experts, w.shared
    r = MoeRouting.choose(h, w)
    rows = r.tile_group.numel() * SEGMENT
    ld = h.stride(0)
    xs = torch.empty(rows, ld, device=h.device, dtype=h.dtype)
    row_of = torch.empty(T * w.top, device=h.device, dtype=torch.int32)
    row_score = torch.empty(rows, device=h.device, dtype=torch.float32)
    _lib.call("ft_moe_gather", h, ld * es, r.expert, r.score, r.pos, r.start, T, w.top, round_up(w.width, 8) * es, xs, ld * es, row_of, row_score, _lib.S())
    gu = torch.empty(rows, 2 * x.fp, device=h.device, dtype=h.dtype)
    grouped_linear(xs, x.gu, r.tile_group, 2 * x.fp, w.width, gu)
    act = gated_act(gu, x.fp, x.limit, w.slope, row_score, r.rows_used, w.form)
    out = torch.empty(rows, round_up(w.width, 8), device=h.device, dtype=h.dtype)
    grouped_linear(act, x.down, r.tile_group, w.width, x.ff, out)
    planes = None
    if s is not None:
        sgu = linear_rows(h, s.gu[0][:, : w.width])
        planes = linear_rows(gated_act(sgu, s.fp, s.limit, w.slope, form=w.form)[:, : s.ff], s.down[0][: w.width, : s.ff], out_f32=True)
        planes = planes.as_strided((1, T, w.width), (0, planes.stride(0), 1))
    return SublayerOutput(planes=planes, rows=out, row_of=row_of, top=w.top)
