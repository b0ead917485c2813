"""Latent attention (keys and values expanded from one small cached vector per token, optionally one rotated key part shared by all heads) on the kernels of
``csrc/kernels/latent_attn.cu``. Queries may come through a latent of their own, a layer may read the latent that an earlier layer cached, and the heads' outputs may be
gated (per element or per head).

Prompts expand keys and values per head with a GEMM and run a tcgen05 flash kernel over ragged sequences; a decode step folds ``W_uk`` into the query
and ``W_uv`` into the output, so that it reads nothing but the cached rows. f32 data takes the folded form everywhere, on a plain kernel.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _lib
from ..errors import InvalidArgument
from .gemm import gemm
from .gqa_attention import GATE_ELEMENT, GATE_NONE
from .moe import linear_rows
from .streams import SublayerOutput, padded_vector, round_up

SMALL_TOKENS = 16
_SMEM_MAX = 232448


@dataclass(frozen=True)
class LatentDims:
    """Sizes of one latent-attention layer: per head ``dim`` plain and ``rot_dim`` (possibly 0) rotated query / key dimensions and ``vdim`` value dimensions; a
    latent of ``rank``. The padded sizes give the layouts the kernels share: projection rows ``heads x [dim8 | rot8] | rank8 | rot8 | gate``, cache rows ``[r16 | rot16]``."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    rank: int
    scale: float
    eps: float
    q_rank: int = 0                      # queries from a normalised latent of this size (without a rotated part)
    own: bool = True                     # the layer has a latent of its own; otherwise it reads an earlier layer's
    gate: int = GATE_NONE                # of the heads' outputs

    @property
    def dim8(self): return round_up(self.dim, 8)
    @property
    def rot8(self): return round_up(self.rot_dim, 8)
    @property
    def v8(self): return round_up(self.vdim, 8)
    @property
    def rank8(self): return round_up(self.rank, 8)
    @property
    def r16(self): return round_up(self.rank, 16)
    @property
    def row(self): return self.r16 + round_up(self.rot_dim, 16)
    @property
    def q_cols(self): return round_up(self.q_rank, 8) if self.q_rank else self.heads * (self.dim8 + self.rot8)
    @property
    def gate_col(self): return self.q_cols + (self.rank8 + self.rot8 if self.own else 0)
    @property
    def gate_cols(self): return 0 if self.gate == GATE_NONE else self.heads * self.v8 if self.gate == GATE_ELEMENT else self.heads
    @property
    def proj_cols(self): return self.gate_col + round_up(self.gate_cols, 8)

    def flash_tile(self) -> int:
        """Query rows per tile of the flash kernel, 0 when these sizes do not fit it."""
        nq, nv = -(-self.dim // 64) + -(-self.rot_dim // 64), -(-self.vdim // 64)
        if nq <= 2 and nv == 1:
            return 128
        for nt, limit in ((2, 2), (1, 4)):
            if nv <= limit and nt * nq * 16384 + 2 * (nq + nv) * 8192 + nt * 16384 + 1280 <= _SMEM_MAX:
                return 128 * nt
        return 0

    def head_tiles(self) -> int:
        """16-head tiles per CTA of the decode kernel (1 or 2), 0 when these sizes do not fit it."""
        per_warp = -(-(self.r16 // 16) // 8)
        for mt in ((2, 1) if self.heads > 16 else (1,)):
            smem = (mt * 16 + 128) * (self.row * 2 + 16) + mt * 16 * 144
            if smem <= _SMEM_MAX - 8192 and per_warp <= (8 if mt == 1 else 4):
                return mt
        return 0

    def decode_supported(self) -> bool:
        fits = max(self.dim * (128 + 4 * SMALL_TOKENS), self.rank * 4, self.q_rank * 4) <= 48 * 1024
        return self.head_tiles() > 0 and fits and SMALL_TOKENS * (2 * round_up(self.rank, 32) + 64) + 64 <= 208 * 1024


@dataclass
class LatentWeights:
    """Packed projections: ``proj`` ``[proj_cols, width]`` (queries or query latent, latent, shared rotated key, gate), ``ukv`` ``[heads * dim8 + heads * v8 (+ 16), rank32]``
    (key, then value expansion of every head), ``out`` ``[width, heads * v8]``, ``norm`` f32; with a query latent its expansion ``uq`` ``[heads * dim8, q_rank]``
    and norm ``q_norm``."""
    dims: LatentDims
    proj: torch.Tensor
    ukv: torch.Tensor
    out: torch.Tensor
    norm: Optional[torch.Tensor]
    uq: Optional[torch.Tensor] = None
    q_norm: Optional[torch.Tensor] = None

    @staticmethod
    def pack(dims: LatentDims, q, dkv, norm, uk, uv, out, device, dtype, dq=None, q_norm=None, gate=None) -> "LatentWeights":
        """With a query latent, ``dq`` projects to it, ``q_norm`` norms it and ``q`` expands it; ``dkv`` and ``norm`` are ``None`` where the latent is an earlier layer's."""
        D, W = dims, out.shape[0]
        H = D.heads
        if (D.q_rank > 0) != (dq is not None) or (D.q_rank and (D.rot_dim or D.gate)) or D.own != (dkv is not None) or (D.gate != GATE_NONE) != (gate is not None):
            raise InvalidArgument("latent attention: weights and sizes must agree on the query latent (which has no rotated part and no gate), on the latent and on the gate")

        def place(rows, cols):
            return torch.zeros(rows, round_up(cols, 32), device=device, dtype=dtype)
        proj, K = place(D.proj_cols, W), q.shape[1]
        head = torch.zeros(H, D.dim8 + D.rot8, K, device=device, dtype=dtype)
        qh = q.to(device, dtype).reshape(H, D.dim + D.rot_dim, K)
        head[:, : D.dim], head[:, D.dim8: D.dim8 + D.rot_dim] = qh[:, : D.dim], qh[:, D.dim:]
        uq = None
        if D.q_rank:
            proj[: D.q_rank, :W] = dq.to(device, dtype)
            uq = place(H * D.dim8, K)
            uq[:, :K] = head.reshape(-1, K)
        else:
            proj[: D.q_cols, :W] = head.reshape(D.q_cols, W)
        if D.own:
            proj[D.q_cols: D.q_cols + D.rank, :W] = dkv[: D.rank].to(device, dtype)
            proj[D.q_cols + D.rank8: D.q_cols + D.rank8 + D.rot_dim, :W] = dkv[D.rank:].to(device, dtype)
        if gate is not None:
            g = gate.to(device, dtype)
            if D.gate == GATE_ELEMENT:
                proj[D.gate_col: D.gate_col + H * D.v8].view(H, D.v8, -1)[:, : D.vdim, :W] = g.reshape(H, D.vdim, W)
            else:
                proj[D.gate_col: D.gate_col + H, :W] = g
        ukv = place(H * (D.dim8 + D.v8) + 16, D.rank)                  # 16 spare rows: the decode kernel reads whole 16-row blocks
        ukv[: H * D.dim8].view(H, D.dim8, -1)[:, : D.dim, : D.rank] = uk.to(device, dtype).reshape(H, D.dim, D.rank)
        ukv[H * D.dim8: H * (D.dim8 + D.v8)].view(H, D.v8, -1)[:, : D.vdim, : D.rank] = uv.to(device, dtype).reshape(H, D.vdim, D.rank)
        wo = place(W, H * D.v8)
        wo[:, : H * D.v8].view(W, H, D.v8)[:, :, : D.vdim] = out.to(device, dtype).reshape(W, H, D.vdim)
        return LatentWeights(D, proj[:, :W], ukv, wo[:, : H * D.v8], padded_vector(norm, device) if D.own else None, uq[:, :K] if D.q_rank else None,
                             padded_vector(q_norm, device) if D.q_rank else None)

    @property
    def uv(self) -> torch.Tensor:
        return self.ukv[self.dims.heads * self.dims.dim8:]


def rotary_pair_tables(max_pos: int, dims: int, base: float, device, scaling: Optional[dict] = None):
    """cos / sin ``[max_pos, dims / 2]`` (f32, angles in f64) of rotations with frequencies ``base ** (-2 i / dims)``, scaled as :func:`rope_inv_freq` describes."""
    from .llama import rope_tables
    return rope_tables(max_pos, dims, base, device, scaling)


def absorb_queries(q: torch.Tensor, w: LatentWeights) -> torch.Tensor:
    """``[rows, heads, row]``: ``W_uk^T q_plain`` and the rotated part of projection rows ``q``, the query form that meets cached rows directly."""
    D, T, f32 = w.dims, q.shape[0], q.dtype == torch.float32
    full = torch.zeros(T, D.heads, D.row, device=q.device, dtype=q.dtype)
    hp = D.dim8 + D.rot8
    heads = q[:, : D.heads * hp].unflatten(1, (D.heads, hp))
    full[:, :, D.r16: D.r16 + D.rot_dim] = heads[:, :, D.dim8: D.dim8 + D.rot_dim]
    if f32:
        _lib.call("ft_gemm_simt", 0, q, w.ukv, full, D.heads, T, D.rank, D.dim, q.stride(0), w.ukv.stride(0), full.stride(0), hp, D.dim8 * w.ukv.stride(0), D.row,
                  0, 0, 1.0, 0.0, _lib.S())
    else:
        for n in range(D.heads):
            gemm(heads[:, n, : D.dim], w.ukv[n * D.dim8: n * D.dim8 + D.dim, : D.rank], b_mn=True, out=full[:, n, : D.rank])
    return full


def expand_values(o: torch.Tensor, w: LatentWeights) -> torch.Tensor:
    """``[rows, heads * v8]`` from latent outputs ``o`` ``[rows, heads, r16]``."""
    D, T = w.dims, o.shape[0]
    out = torch.zeros(T, D.heads * D.v8, device=o.device, dtype=o.dtype)
    if o.dtype == torch.float32:
        _lib.call("ft_gemm_simt", 0, o, w.uv, out, D.heads, T, D.vdim, D.rank, o.stride(0), w.uv.stride(0), out.stride(0), D.r16, D.v8 * w.uv.stride(0), D.v8, 0, 1,
                  1.0, 0.0, _lib.S())
    else:
        for n in range(D.heads):
            gemm(o[:, n, : D.rank], w.uv[n * D.v8: n * D.v8 + D.vdim, : D.rank], out=out[:, n * D.v8: n * D.v8 + D.vdim])
    return out


def latent_context(dims: LatentDims, batch, device, dtype) -> torch.Tensor:
    """Room for the latent rows of the batch's sequences, earlier tokens included, one after another."""
    return torch.empty(batch.ctx_total, dims.row, device=device, dtype=dtype)


def latent_attention_rows(h: torch.Tensor, w: LatentWeights, batch, cache: torch.Tensor, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor],
                          ctx: Optional[torch.Tensor] = None) -> SublayerOutput:
    """Attention of a ragged batch of new tokens (prompts, portions of prompts, single tokens). ``batch`` holds the row tables of
    :class:`~ferrotorch_b200.models.serving.RowBatch`; ``cache`` is the page storage ``[pages, 16, row]`` of the layer that has the latent. ``ctx``
    (:func:`latent_context`; bf16 only): filled by a layer with a latent of its own, read by one that takes an earlier layer's."""
    D, T = w.dims, h.shape[0]
    f32 = h.dtype == torch.float32
    q = linear_rows(h, w.proj)
    flash = not f32 and batch.tiles_for(D) is not None
    if flash and ctx is None:
        if not D.own:
            raise InvalidArgument("latent attention: an earlier layer's latent rows are needed")
        ctx = latent_context(D, batch, h.device, h.dtype)
    fill = ctx is not None and D.own
    _lib.call("ft_latent_prep", q, q.stride(0), T, D.heads, D.dim, D.rot_dim, D.rank, D.q_rank, w.q_norm, w.norm, D.eps, batch.positions, cos, sin, batch.slots,
              batch.ctx_rows if fill else None, cache if D.own else None, ctx if fill else None, int(f32), _lib.S())
    if fill and batch.past_slots is not None:
        _lib.call("ft_latent_ctx_gather", cache, ctx, D.row * 2, batch.past_slots, batch.past_rows, batch.past_slots.numel(), _lib.S())
    gate = q[:, D.gate_col:] if D.gate else None
    gating = (gate, 0 if gate is None else gate.stride(0), D.gate)
    if D.q_rank:
        q = linear_rows(q[:, : D.q_rank], w.uq)
    if flash:
        kv = linear_rows(ctx[:, : D.rank], w.ukv[: D.heads * (D.dim8 + D.v8), : D.rank])
        a = torch.empty(T, D.heads * D.v8, device=h.device, dtype=h.dtype)
        tiles = batch.tiles_for(D)
        _lib.call("ft_latent_flash", q, q.stride(0), T, kv, kv.stride(0), ctx[:, D.r16:] if D.rot_dim else None, D.row, batch.ctx_total, tiles, tiles.shape[0], D.heads, D.dim, D.rot_dim,
                  D.vdim, D.scale, *gating, a, a.stride(0), _lib.S())
    else:
        full = absorb_queries(q, w)
        o = torch.empty(T, D.heads, D.r16, device=h.device, dtype=h.dtype)
        for r0 in range(0, T, 32768):
            r1 = min(T, r0 + 32768)
            _lib.call("ft_latent_rows", full[r0:r1], cache, batch.block_table, batch.block_table.shape[1], batch.seq_of[r0:r1], batch.positions[r0:r1], r1 - r0,
                      D.heads, D.rot_dim, D.rank, D.scale, o[r0:r1], int(f32), _lib.S())
        a = expand_values(o, w)
        if D.gate:
            _lib.call("ft_latent_gate", a, a.stride(0), *gating, T, D.heads, D.v8, int(f32), _lib.S())
    y = linear_rows(a, w.out, out_f32=True)
    return SublayerOutput(planes=y.as_strided((1, T, y.shape[1]), (0, y.stride(0), 1)))


class LatentDecodeBuffers:
    """Scratch of the decode kernels for one layer size (shared by layers of the same size, which run one after another)."""

    def __init__(self, dims: LatentDims, max_batch: int, max_tokens: int, device, splits: Optional[int] = None):
        D = dims
        self.mt = D.head_tiles()
        self.tiles = -(-D.heads // (16 * self.mt))
        # by batch size: one CTA per SM (the ring takes most of its shared memory), at least one 64-row chunk per split at the longest sequence
        self.splits = [splits or max(1, min(64, 148 // (b * self.tiles), -(-max_tokens // 64))) for b in range(1, max_batch + 1)]
        self.q = torch.zeros(SMALL_TOKENS, D.heads, D.row, device=device, dtype=torch.bfloat16)
        self.lat = torch.zeros(SMALL_TOKENS, D.heads, D.r16, device=device, dtype=torch.bfloat16)
        self.ws = torch.zeros(max(b * n for b, n in enumerate(self.splits, 1)) * self.tiles * self.mt * 16 * (D.r16 + 4), device=device)
        self.attn = torch.zeros(SMALL_TOKENS, D.heads * D.v8, device=device, dtype=torch.bfloat16)
        self.gate = torch.zeros(SMALL_TOKENS, max(D.gate_cols, 1), device=device)
        self.cq = torch.zeros(SMALL_TOKENS, round_up(max(D.q_rank, 1), 8), device=device, dtype=torch.bfloat16)[:, : D.q_rank]


def latent_attention_decode(planes: torch.Tensor, splits: int, w: LatentWeights, b: LatentDecodeBuffers, state, cache: torch.Tensor, cos, sin, B: int,
                            expand=None) -> torch.Tensor:
    """One token per sequence from the split-K planes of the projection: returns the attention output rows ``[16, heads * v8]`` (bf16, in ``b``). ``expand``: the split-K
    product of ``w.uq`` where queries come through a latent."""
    D, S = w.dims, _lib.S()
    bt, mb, nsplit = state.block_table, state.block_table.shape[1], b.splits[B - 1]
    own, gate = cache if D.own else None, b.gate if D.gate else None
    if D.q_rank:
        _lib.call("ft_latent_decode_norms", planes, splits, planes.stride(1), planes.stride(0), B, D.q_rank, D.rank, w.q_norm, w.norm, D.eps, state.positions, bt, mb,
                  b.cq, b.cq.stride(0), own, S)
        expand(b.cq)
        planes, splits, own = expand.planes, expand.splits, None
    _lib.call("ft_latent_decode_prep", planes, splits, planes.stride(1), planes.stride(0), B, D.heads, D.dim, D.rot_dim, D.rank, w.ukv, w.ukv.stride(0), w.norm, D.eps,
              state.positions, cos, sin, bt, mb, b.q, own, D.gate_cols, gate, S)
    _lib.call("ft_latent_decode", b.q, cache, bt, mb, state.seq_lens, B, D.heads, D.rot_dim, D.rank, D.scale, nsplit, b.mt, b.ws, S)
    _lib.call("ft_latent_combine", b.ws, B, D.heads, D.rank, nsplit, b.mt, b.lat, S)
    _lib.call("ft_skinny_heads", b.lat, b.lat.stride(0), b.lat.stride(1), w.uv, w.uv.stride(0), D.v8 * w.uv.stride(0), B, D.heads, D.vdim, D.rank, b.attn,
              b.attn.stride(0), D.v8, gate, D.gate_cols, D.v8 if D.gate == GATE_ELEMENT else 1, int(D.gate == GATE_ELEMENT), S)
    return b.attn
