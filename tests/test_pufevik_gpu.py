"""Pufevik on the device against the plain f64 evaluation in ``pufevik_oracle``: every mechanism by itself, then prompts, portions of prompts, decoding, batches, reuse of
pages and state slots, and generation."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import pufevik_oracle as O
from ferrotorch_b200.errors import InvalidArgument
from ferrotorch_b200.models import (DecodeState, GenerationConfig, PufevikConfig, PufevikModel, RandomPufevikWeights, RowBatch, ServingEngine, SpecDecodeConfig, StepEntry,
                                    beam_search, generate, speculative_generate)
from ferrotorch_b200.nn import PagedRowCache, PagePool, StateSlots
from ferrotorch_b200.ops import (DenseGatedWeights, GqaDecodeBuffers, GqaDims, GqaWeights, MemoryDims, MemoryWeights, SublayerOutput, dense_gated_rows, gated_act_planes,
                                 gated_act_rows, gqa_attention_decode, gqa_attention_rows, matrix_memory_decode, matrix_memory_rows, pack_head_columns, residual_embed,
                                 residual_update)
from ferrotorch_b200.ops.gqa_attention import GATE_ELEMENT, GATE_HEAD, GATE_NONE
from ferrotorch_b200.ops.latent_attention import rotary_pair_tables
from ferrotorch_b200.ops.streams import padded_vector, round_up

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
TOL = {F32: 5e-6, BF16: 2e-2}


def dev(a, dtype=F32):
    return torch.as_tensor(np.asarray(a, dtype=np.float32)).cuda().to(dtype)


def rounded(a, dtype):
    """f64 values of the device copy (so that input rounding is not part of the error)."""
    return dev(a, dtype).double().cpu().numpy()


def padded(a, dtype, multiple=8):
    t = dev(a, dtype)
    buf = torch.full((t.shape[0], round_up(t.shape[1], multiple)), float("nan"), device="cuda", dtype=dtype)
    buf[:, : t.shape[1]] = t
    return buf[:, : t.shape[1]]


def rel(got, want):
    """Largest row error relative to the rms of the reference."""
    g, w = got.double().cpu().numpy(), np.asarray(want, dtype=np.float64)
    assert g.shape == w.shape and np.isfinite(g).all()
    return float(np.sqrt(((g - w) ** 2).mean(-1)).max() / (np.sqrt((w ** 2).mean()) + 1e-30))


def split_planes(rows, n, rng, pad=16):
    """f32 rows as ``n`` planes of ``pad`` rows that sum to them."""
    parts = rng.standard_normal((n, *rows.shape))
    parts[-1] = rows - parts[:-1].sum(0)
    out = torch.full((n, pad, round_up(rows.shape[1], 4)), float("nan"), device="cuda")
    out[:, : rows.shape[0], : rows.shape[1]] = dev(parts)
    return out


# -- residual and activation -------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width", [(1, 5), (3, 2052), (16, 640), (300, 68), (2, 9001)])
def test_residual_start_update_and_end(dtype, rows, width):
    rng = np.random.default_rng(rows)
    table, ids = rounded(rng.standard_normal((11, width)), dtype), rng.integers(0, 11, rows)
    ld = round_up(width, 8)
    x = torch.full((rows, ld), float("nan"), device="cuda")
    h = torch.full((rows, ld), float("nan"), device="cuda", dtype=dtype)[:, :width]
    residual_embed(torch.as_tensor(ids).cuda(), padded(table, dtype), 2.5, x, h, rows)
    want = 2.5 * table[ids]
    assert rel(x[:, :width], want) < 1e-6 and rel(h, want) < TOL[dtype]
    w, last = rng.standard_normal(width), rng.standard_normal(width)
    for n, final, store in ((1, False, True), (6, True, False), (5, True, True)):
        y = 0.02 * rng.standard_normal((rows, width))
        planes = split_planes(y, n, rng, pad=rows + 1)
        before = x.clone()
        residual_update(x, SublayerOutput(planes=planes), padded_vector(dev(w), "cuda"), 1e-3, h, rows, width, padded_vector(dev(last), "cuda") if final else None, store)
        new = want + O.rms_norm(planes[:, :rows, :width].double().sum(0).cpu().numpy(), dev(w).double().cpu().numpy(), 1e-3)
        assert rel(h, O.rms_norm(new, dev(last).double().cpu().numpy(), 1e-3) if final else new) < (1e-5 if dtype == F32 else 1e-2)
        if store:
            assert rel(x[:, :width], new) < 5e-6
            want = x[:, :width].double().cpu().numpy()
        else:
            assert torch.equal(x[:, :width], before[:, :width])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width,ff", [(24, 8), (40, 33), (64, 700)])
def test_gated_feed_forward(dtype, width, ff):
    rng = np.random.default_rng(ff)
    W = {k: rounded(rng.standard_normal(s) / s[1] ** 0.5 * 1.5, dtype) for k, s in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))}
    w = DenseGatedWeights.pack(*(torch.tensor(W[k]) for k in ("gate", "up", "down")), "cuda", dtype)
    for rows in (1, 5, 130):
        h = rounded(2.0 * rng.standard_normal((rows, width)), dtype)
        got = dense_gated_rows(padded(h, dtype), w).planes[0]
        assert rel(got, O.feed_forward(h, W)) < (1e-5 if dtype == F32 else 2e-2)
    gu = rounded(3.0 * rng.standard_normal((7, 2 * w.fp)), F32)
    blocks = gu.reshape(7, w.fp // 8, 2, 8)
    g, u = blocks[:, :, 0].reshape(7, -1), blocks[:, :, 1].reshape(7, -1)
    for act, f in (("gelu_tanh", O.gelu_tanh), ("silu", lambda z: z * O.sigmoid(z))):
        assert rel(gated_act_rows(dev(gu, dtype), w.fp, act), f(rounded(g, dtype)) * rounded(u, dtype)) < (2e-6 if dtype == F32 else 1e-2)
        out = torch.zeros(16, w.fp, device="cuda", dtype=BF16)
        gated_act_planes(split_planes(gu, 3, rng), 3, 7, w.fp, act, out)
        assert rel(out[:7], f(g) * u) < 1e-2 and not out[7:].any()


# -- attention ---------------------------------------------------------------------------------------------------------------------------
class AttentionRig:
    """One attention layer fed with projection rows: weights, a page cache full of other sequences' leftovers, and the reference."""

    def __init__(self, D, dtype, seed=0, sink=None, mix=None, tokens=2048):
        self.D, self.dtype, self.rng = D, dtype, np.random.default_rng(seed)
        nq, nk = (D.heads * D.dim, D.kv_heads * D.dim) if D.whole_norm else (D.dim, D.dim)
        self.qn, self.kn = (rounded(1.0 + 0.2 * self.rng.standard_normal(n), F32) for n in (nq, nk))
        self.sink, self.mix = sink, mix
        self.base = 700.0
        self.w = GqaWeights.pack(D, torch.tensor(self.qn), torch.tensor(self.kn), "cuda", None if sink is None else torch.tensor(sink), None if mix is None else torch.tensor(mix))
        self.tables = rotary_pair_tables(tokens, D.rot_dims, self.base, "cuda")
        self.pool = PagePool(tokens // 16 + 8, 16)
        self.rng.shuffle(self.pool.free)
        self.cache = PagedRowCache(self.pool, [D.row], "cuda", dtype)
        self.cache.rows[0].normal_()
        self.blocks = tokens // 16

    def projections(self, n):
        """Raw queries, keys, values and gates of ``n`` tokens, rounded to the data type, and earlier values to mix in."""
        D = self.D
        r = lambda *s: rounded(self.rng.standard_normal((n, *s)), self.dtype)
        gate = r(D.heads, D.vdim) if D.gate == GATE_ELEMENT else rounded(self.rng.standard_normal((n, D.heads)), F32)
        return dict(q=r(D.heads, D.dim), k=r(D.kv_heads, D.dim), v=r(D.kv_heads, D.vdim), gate=gate, first=r(D.kv_heads, D.vdim))

    def rows(self, P, lo, hi):
        """Device projection rows ``[tokens, qkv (+ element gate)]`` in the kernels' padding."""
        D = self.D
        cols = [pack_head_columns(torch.tensor(P[k][lo:hi]).flatten(1), n, s, "cuda", self.dtype)
                for k, n, s in (("q", D.heads, D.dim), ("k", D.kv_heads, D.dim), ("v", D.kv_heads, D.vdim))]
        if D.gate == GATE_ELEMENT:
            cols.append(pack_head_columns(torch.tensor(P["gate"][lo:hi]).flatten(1), D.heads, D.vdim, "cuda", self.dtype))
        return torch.cat(cols, 1).contiguous()

    def first_rows(self, P, lo, hi, dtype):
        return None if self.mix is None else pack_head_columns(torch.tensor(P["first"][lo:hi]).flatten(1), self.D.kv_heads, self.D.vdim, "cuda", dtype).contiguous()

    def reference(self, P):
        D, n = self.D, P["q"].shape[0]

        def norm(x, w):
            return O.rms_norm(x.reshape(n, -1), w, D.eps).reshape(x.shape) if D.whole_norm else O.rms_norm(x, w, D.eps)
        q, k = (O.rotate_first_pairs(norm(P[a], w), np.arange(n), D.rot_dims, self.base) for a, w in (("q", self.qn), ("k", self.kn)))
        v = P["v"] if self.mix is None else (1 - self.mix) * P["v"] + self.mix * P["first"]
        o = O.attend(q, k, v, D.scale, D.window or None, self.sink)
        if D.gate == GATE_ELEMENT:
            o = o * O.sigmoid(P["gate"])
        elif D.gate == GATE_HEAD:
            o = o * O.sigmoid(P["gate"])[:, :, None]
        return o * D.out_scale

    def heads_of(self, out):
        return out.view(out.shape[0], self.D.heads, self.D.v16)[..., : self.D.vdim]

    def open(self, ids):
        for s in ids:
            self.cache.add_sequence(s)

    def step(self, parts):
        """``parts``: {sequence: (projections, first token, end)}; returns the output heads of the new tokens."""
        entries = [StepEntry(s, [0] * (hi - lo)) for s, (_, lo, hi) in parts.items()]
        for e in entries:
            self.cache.reserve(e.id, self.cache.lengths[e.id] + len(e.tokens))
        batch = RowBatch(entries, self.cache, torch.device("cuda"), self.blocks)
        x = torch.cat([self.rows(*p) for p in parts.values()])
        gate = None
        if self.D.gate == GATE_ELEMENT:
            gate = x[:, self.D.qkv_cols:]
        elif self.D.gate == GATE_HEAD:
            gate = dev(np.concatenate([p["gate"][lo:hi] for p, lo, hi in parts.values()]))
        first = None if self.mix is None else torch.cat([self.first_rows(*p, self.dtype) for p in parts.values()])
        out = torch.full((x.shape[0], self.D.out_cols), float("nan"), device="cuda", dtype=self.dtype)
        gqa_attention_rows(x, self.w, batch, self.cache.rows[0], *self.tables, gate, out, first)
        for e in entries:
            self.cache.lengths[e.id] += len(e.tokens)
        return self.heads_of(out)

    def decode(self, parts, splits=None):
        """One token per sequence: {sequence: (projections, token)}."""
        B, D = len(parts), self.D
        state = DecodeState("cuda", self.blocks)
        ids = list(parts)
        for s in ids:
            self.cache.reserve(s, self.cache.lengths[s] + 1)
        state.load([0] * B, [self.cache.lengths[s] for s in ids], self.cache.block_table(ids, self.blocks))
        x = torch.cat([self.rows(p, t, t + 1) for p, t in parts.values()]).double().cpu().numpy()
        if D.gate == GATE_HEAD:
            x = np.concatenate([x, np.concatenate([p["gate"][t: t + 1] for p, t in parts.values()])], 1)
        planes = split_planes(x, 3, self.rng)
        b = GqaDecodeBuffers(D, 16, self.blocks * 16, "cuda", splits)
        first = None
        if self.mix is not None:
            first = torch.zeros(16, D.kv_heads * D.v16, device="cuda")
            first[:B] = torch.cat([self.first_rows(p, t, t + 1, F32) for p, t in parts.values()])
        out = torch.zeros(16, D.out_cols, device="cuda", dtype=BF16)
        keep = torch.zeros(16, D.kv_heads * D.v16, device="cuda")
        for _ in range(2):                                  # the second run finds the counters as the first one left them
            gqa_attention_decode(planes, 3, self.w, b, state, self.cache.rows[0], *self.tables, B, D.qkv_cols, out, keep if first is None else None, first)
        if first is None:
            v = np.concatenate([p["v"][t: t + 1] for p, t in parts.values()])
            assert rel(keep.view(16, D.kv_heads, D.v16)[:B, :, : D.vdim].flatten(1), v.reshape(B, -1)) < 1e-5
        for s in ids:
            self.cache.lengths[s] += 1
        assert not b.counters.any() and not out[B:].any()
        return self.heads_of(out)[:B]


def dims(heads, kv_heads, dim, vdim, rot, window=0, whole=False, gate=GATE_NONE, scale=None, out_scale=1.0):
    return GqaDims(heads, kv_heads, dim, vdim, rot, scale or 1.3 * dim ** -0.5, 1e-4, window, whole, gate, out_scale)


CASES = {
    "one head": (dims(1, 1, 8, 8, 0), {}),
    "group of four, element gate, mixed values": (dims(8, 2, 48, 40, 24, gate=GATE_ELEMENT), dict(mix=0.35)),
    "group of three, window, sink, head gate": (dims(6, 2, 80, 96, 20, window=50, whole=True, gate=GATE_HEAD, out_scale=0.6), dict(sink=np.array([2.0, -1.0, 0.5, 4.0, -6.0, 1.0]))),
    "group of five, odd sizes": (dims(5, 1, 23, 11, 22, window=7, whole=True), dict(sink=np.linspace(-2, 3, 5))),
    "many heads of one key": (dims(40, 1, 64, 64, 64, gate=GATE_HEAD), {}),
    "wide heads": (dims(4, 4, 128, 128, 128, window=130, gate=GATE_ELEMENT), {}),
    "wider keys": (dims(2, 1, 200, 60, 100, whole=True), {}),
    "wider values": (dims(2, 2, 64, 250, 2), {}),
    "window of one": (dims(4, 2, 32, 16, 4, window=1), dict(sink=np.array([0.0, 1.0, -1.0, 2.0]))),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", CASES)
def test_attention_of_ragged_prompts_and_portions(case, dtype):
    D, kw = CASES[case]
    rig = AttentionRig(D, dtype, 1, **kw)
    P = {s: rig.projections(n) for s, n in (("a", 150), ("b", 1), ("c", 293))}
    want = {s: rig.reference(p) for s, p in P.items()}
    rig.open(P)
    cuts = {"a": [0, 2, 71, 150], "b": [0, 1, 1, 1], "c": [0, 129, 131, 293]}
    got = {s: [] for s in P}
    for i in range(3):
        parts = {s: (P[s], c[i], c[i + 1]) for s, c in cuts.items() if c[i + 1] > c[i]}
        out = rig.step(parts)
        at = 0
        for s, (_, lo, hi) in parts.items():
            got[s].append(out[at: at + hi - lo])
            at += hi - lo
    for s in P:
        assert rel(torch.cat(got[s]).flatten(1), want[s].reshape(len(want[s]), -1)) < TOL[dtype] * (2 if dtype == F32 else 1), s


@pytest.mark.parametrize("splits", [None, 1, 7])
@pytest.mark.parametrize("case", CASES)
def test_attention_decode_matches_the_whole_sequence(case, splits):
    D, kw = CASES[case]
    assert D.decode_supported()
    rig = AttentionRig(D, BF16, 2, **kw)
    lens = {"a": 0, "b": 15, "c": 16, "d": 200, "e": 64}
    P = {s: rig.projections(n + 3) for s, n in lens.items()}
    want = {s: rig.reference(p) for s, p in P.items()}
    rig.open(P)
    rig.step({s: (P[s], 0, n) for s, n in lens.items() if n})
    for t in range(3):
        got = rig.decode({s: (P[s], n + t) for s, n in lens.items()}, splits)
        assert rel(got.flatten(1), np.stack([want[s][n + t].reshape(-1) for s, n in lens.items()])) < 2e-2


@pytest.mark.parametrize("heads,kv_heads,window", [(4, 1, 1), (4, 1, 16), (6, 2, 37), (8, 1, 64), (3, 3, 100), (8, 1, 129), (4, 1, 0)])
@pytest.mark.parametrize("target", [0, 15, 16, 63, 64, 130])
def test_one_key_stands_out_until_it_leaves_the_window(heads, kv_heads, window, target):
    """One key meets every query with a score far above all others: its value is the output exactly while it is visible. In prompts, portions and decoding, around
    page, block and window borders."""
    D = GqaDims(heads, kv_heads, 32, 16, 8, 0.6, 1e-6, window, False, GATE_NONE, 1.0)
    rig = AttentionRig(D, BF16, target)
    rig.qn[:] = 1.0
    rig.kn[:] = 1.0
    rig.w = GqaWeights.pack(D, torch.tensor(rig.qn), torch.tensor(rig.kn), "cuda")
    n = 270
    P = rig.projections(n)
    P["q"][:] = 0.0
    P["q"][..., 31] = 1.0                                   # beyond the rotated dimensions
    P["k"][..., 31] = 0.0
    P["k"][target] = 0.0
    P["k"][target, :, 31] = 1.0
    want = rig.reference(P)
    seen = [i for i in range(n) if target <= i and (window == 0 or i - target < window)]
    for i in seen:
        assert np.abs(want[i] - np.repeat(P["v"][target], heads // kv_heads, 0)).max() < 1e-3
    rig.open(["whole", "parts", "steps"])
    assert rel(rig.step({"whole": (P, 0, n)}).flatten(1), want.reshape(n, -1)) < 1e-2
    got = [rig.step({"parts": (P, lo, hi)}) for lo, hi in ((0, 66), (66, 68), (68, 200), (200, n))]
    assert rel(torch.cat(got).flatten(1), want.reshape(n, -1)) < 1e-2
    edge = target + (window or 40)
    lo, hi = max(0, edge - 3), min(n, edge + 4)
    if lo:
        rig.step({"steps": (P, 0, lo)})
    for t in range(lo, hi):
        assert rel(rig.decode({"steps": (P, t)}).flatten(1), want[t].reshape(1, -1)) < 1e-2, t


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window", [0, 9])
def test_sink_takes_its_share_from_the_first_token_on(dtype, window):
    """All scores equal: a query that sees n keys gives each 1 / (n + e^sink)."""
    D = GqaDims(4, 2, 16, 16, 0, 0.5, 1e-6, window)
    sink = np.array([-30.0, 0.0, 2.0, 25.0])
    rig = AttentionRig(D, dtype, 3, sink=sink)
    P = rig.projections(40)
    P["q"][:], P["v"][:] = 0.0, 1.0
    n = np.minimum(np.arange(40) + 1, window or 40)
    want = n[:, None] / (n[:, None] + np.exp(sink)[None, :])
    rig.open("ab")
    got = rig.step({"a": (P, 0, 40)}).double().cpu().numpy()
    assert np.abs(got - want[:, :, None]).max() < (1e-6 if dtype == F32 else 1e-2)
    if dtype == BF16:
        for t in range(12):
            assert np.abs(rig.decode({"b": (P, t)}).double().cpu().numpy()[0] - want[t][:, None]).max() < 1e-2


# -- matrix memory -----------------------------------------------------------------------------------------------------------------------
class MemoryRig:
    def __init__(self, D, dtype, seed=0, slots=8, bias=(-1.0, 3.0)):
        self.D, self.dtype, self.rng = D, dtype, np.random.default_rng(seed)
        self.bi, self.bf = (rounded(m + self.rng.standard_normal(D.heads), F32) for m in bias)
        self.norm = rounded(1.0 + 0.2 * self.rng.standard_normal(D.heads * D.vdim), F32)
        self.w = MemoryWeights.pack(D, *(torch.tensor(t) for t in (self.bi, self.bf, self.norm)), "cuda")
        self.states = StateSlots(slots, [D.state_size], "cuda")
        self.states.data[0].fill_(float("nan"))              # what a sequence finds in its slot must not matter
        self.cache = PagedRowCache(PagePool(400, 16), [8], "cuda", dtype, self.states)

    def projections(self, n, gate_scale=2.0):
        D = self.D
        r = lambda *s: rounded(self.rng.standard_normal((n, *s)), self.dtype)
        return dict(q=r(D.heads, D.dim), k=r(D.heads, D.dim), v=r(D.heads, D.vdim), g=r(D.heads, D.vdim), i=rounded(gate_scale * self.rng.standard_normal((n, D.heads)), F32),
                    f=rounded(gate_scale * self.rng.standard_normal((n, D.heads)), F32))

    def reference(self, P):
        """Outputs ``[tokens, heads, vdim]`` and the final states."""
        D, n = self.D, P["q"].shape[0]

        def soft(z):
            return D.cap * np.tanh(z / D.cap)
        i, f = soft(P["i"] + self.bi), -np.logaddexp(0.0, -soft(P["f"] + self.bf))
        o, last = np.zeros((n, D.heads, D.vdim)), []
        for h in range(D.heads):
            y, st = O.matrix_memory(P["q"][:, h] * D.dim ** -0.5, P["k"][:, h], P["v"][:, h], i[:, h], f[:, h])
            o[:, h] = O.rms_norm(y, self.norm.reshape(D.heads, -1)[h], D.eps)
            last.append(st)
        return o * O.sigmoid(P["g"]) * D.out_scale, last

    def rows(self, P, lo, hi):
        D = self.D
        x = torch.cat([pack_head_columns(torch.tensor(P[k][lo:hi]).flatten(1), D.heads, s, "cuda", F32) for k, s in (("q", D.dim), ("k", D.dim), ("v", D.vdim), ("g", D.vdim))], 1)
        gates = torch.full((hi - lo, 2 * D.h8), float("nan"), device="cuda")
        gates[:, : D.heads], gates[:, D.h8: D.h8 + D.heads] = dev(P["i"][lo:hi]), dev(P["f"][lo:hi])
        return x, gates

    def heads_of(self, out):
        return out.view(out.shape[0], self.D.heads, self.D.v16)[..., : self.D.vdim].flatten(1)

    def step(self, parts, walk=None):
        entries = [StepEntry(s, [0] * (hi - lo)) for s, (_, lo, hi) in parts.items()]
        for e in entries:
            self.cache.reserve(e.id, self.cache.lengths[e.id] + len(e.tokens))
        batch = RowBatch(entries, self.cache, torch.device("cuda"), 100)
        x, gates = (torch.cat(t) for t in zip(*(self.rows(*p) for p in parts.values())))
        out = torch.full((x.shape[0], self.D.out_cols), float("nan"), device="cuda", dtype=self.dtype)
        matrix_memory_rows(x.to(self.dtype), gates, self.w, batch, self.states.data[0], out, walk)
        for e in entries:
            self.cache.lengths[e.id] += len(e.tokens)
        return self.heads_of(out)

    def decode(self, parts):
        B = len(parts)
        state = DecodeState("cuda", 4)
        state.load([0] * B, [self.cache.lengths[s] for s in parts], torch.zeros(B, 4, dtype=torch.int32), [self.states.slot[s] for s in parts])
        x = torch.cat([torch.cat(self.rows(p, t, t + 1), 1) for p, t in parts.values()])
        x[x.isnan()] = 7.0
        planes = split_planes(np.concatenate([np.full((B, 4), 9.0), x.double().cpu().numpy()], 1), 3, self.rng)
        out = torch.zeros(16, self.D.out_cols, device="cuda", dtype=BF16)
        matrix_memory_decode(planes, 3, self.w, state, self.states.data[0], B, 4, 4 + self.D.proj_cols, out)
        for s in parts:
            self.cache.lengths[s] += 1
        assert not out[B:].any()
        return self.heads_of(out)[:B]

    def state(self, s):
        """``(S, n, m)`` per head."""
        D = self.D
        flat = self.states.data[0][self.states.slot[s]].view(D.heads, -1).double().cpu().numpy()
        nS = D.d16 * D.v16
        return [(f[:nS].reshape(D.d16, D.v16)[: D.dim, : D.vdim], f[nS: nS + D.dim], f[nS + D.d16]) for f in flat]


def state_error(got, want):
    e = 0.0
    for (S, n, m), (S0, n0, m0) in zip(got, want):
        assert abs(m - m0) < 1e-4
        e = max(e, np.abs(S - S0).max() / np.abs(S0).max(), np.abs(n - n0).max() / np.abs(n0).max())
    return e


MEMORIES = [MemoryDims(2, 16, 16, 5.0, 1e-5), MemoryDims(3, 24, 40, 8.0, 1e-4, 0.5), MemoryDims(1, 128, 96, 15.0, 1e-6), MemoryDims(2, 144, 200, 4.0, 1e-6), MemoryDims(9, 5, 3, 2.0, 1e-3),
            MemoryDims(1, 256, 70, 12.0, 1e-6)]


@pytest.mark.parametrize("form", ["f32", "walk", "tokens"])
@pytest.mark.parametrize("D", MEMORIES, ids=lambda d: f"{d.heads}-{d.dim}-{d.vdim}")
def test_matrix_memory_of_prompts_and_portions(D, form):
    """Ragged portions, down to one token, against the recurrence; the state carried to the next portion is exact to 32-bit rounding (the walk's products take
    f32 factors as pairs of bf16 numbers)."""
    dtype = F32 if form == "f32" else BF16
    rig = MemoryRig(D, dtype, 5)
    P = {"a": rig.projections(200), "b": rig.projections(3), "c": rig.projections(65)}
    want = {s: rig.reference(p) for s, p in P.items()}
    for s in P:
        rig.cache.add_sequence(s)
    got = {s: [] for s in P}
    cuts = {"a": [0, 2, 130, 200], "b": [0, 1, 3, 3], "c": [0, 63, 64, 65]}
    for i in range(3):
        parts = {s: (P[s], c[i], c[i + 1]) for s, c in cuts.items() if c[i + 1] > c[i]}
        out = rig.step(parts, None if form == "f32" else form == "walk")
        at = 0
        for s, (_, lo, hi) in parts.items():
            got[s].append(out[at: at + hi - lo])
            at += hi - lo
    for s in P:
        assert rel(torch.cat(got[s]), want[s][0].reshape(len(want[s][0]), -1)) < (2e-5 if form == "f32" else 2e-2), s
        assert state_error(rig.state(s), want[s][1]) < (5e-6 if form != "walk" else 5e-5), s


@pytest.mark.parametrize("D", MEMORIES[:4], ids=lambda d: f"{d.heads}-{d.dim}-{d.vdim}")
def test_long_prompts_walk_in_segments(D):
    """Several segments at the same time, from a fresh state and from a carried one, beside a short sequence."""
    rig = MemoryRig(D, BF16, 6)
    P, Q = rig.projections(1300), rig.projections(70)
    for s in "pq":
        rig.cache.add_sequence(s)
    want, last = rig.reference(P)
    a = rig.step({"p": (P, 0, 700)})
    b = rig.step({"q": (Q, 0, 70), "p": (P, 700, 1300)})
    rig.cache.reserve("p", 1900)
    batch = RowBatch([StepEntry("p", [0] * 600)], rig.cache, torch.device("cuda"), 130)
    assert batch.memory_plan(D.heads * -(-D.v16 // 128)).scratch > 1
    assert rel(torch.cat([a, b[70:]]), want.reshape(1300, -1)) < 2e-2 and state_error(rig.state("p"), last) < 5e-5
    assert rel(b[:70], rig.reference(Q)[0].reshape(70, -1)) < 2e-2


@pytest.mark.parametrize("bias,scale", [((6.0, -6.0), 4.0), ((-6.0, 8.0), 1.0), ((0.0, 0.0), 30.0)])
@pytest.mark.parametrize("form", ["f32", "walk", "decode"])
def test_gates_at_their_limits(bias, scale, form):
    """Input gates far above the running maximum, states that fade within a few tokens, states that are kept for good."""
    D = MemoryDims(2, 16, 24, 9.0, 1e-6)
    rig = MemoryRig(D, F32 if form == "f32" else BF16, 7, bias=bias)
    P = rig.projections(150, scale)
    want, last = rig.reference(P)
    rig.cache.add_sequence("s")
    got = torch.cat([rig.decode({"s": (P, t)}) for t in range(150)]) if form == "decode" else rig.step({"s": (P, 0, 150)})
    assert rel(got, want.reshape(150, -1)) < (5e-4 if form == "f32" else 2e-2) and state_error(rig.state("s"), last) < 1e-4


@pytest.mark.parametrize("D", MEMORIES + [MemoryDims(1, 400, 300, 6.0, 1e-6), MemoryDims(1, 32, 600, 6.0, 1e-6)], ids=lambda d: f"{d.heads}-{d.dim}-{d.vdim}")
def test_matrix_memory_decode(D):
    """Fresh sequences and ones with a prompt behind them; slots that are freed and used again."""
    rig = MemoryRig(D, BF16, 8, slots=5)
    for wave in range(2):
        P = {f"{wave}{i}": rig.projections(n + 4) for i, n in enumerate((0, 1, 80, 64))}
        lens = {s: len(p["q"]) - 4 for s, p in P.items()}
        want = {s: rig.reference(p) for s, p in P.items()}
        for s in P:
            rig.cache.add_sequence(s)
        rig.step({s: (P[s], 0, n) for s, n in lens.items() if n})
        for t in range(4):
            got = rig.decode({s: (P[s], n + t) for s, n in lens.items()})
            assert rel(got, np.stack([want[s][0][n + t].reshape(-1) for s, n in lens.items()])) < 1e-2
        for s in P:
            assert state_error(rig.state(s), want[s][1]) < 5e-5
            rig.cache.free_sequence(s)
    assert rig.states.num_free() == 5


# -- the model ---------------------------------------------------------------------------------------------------------------------------
MODELS = {
    "plain": dict(seed=1, kinds="pap"),
    "attention only, no mixing": dict(seed=2, kinds="aa", v_mix=False, heads=6, kv_heads=3, vdim=16),
    "side by side only": dict(seed=3, kinds="pp", window=9, left_scale=1.3, right_scale=1.0),
    "odd sizes": dict(seed=4, kinds="apaap", vocab=101, width=52, ff=37, heads=5, kv_heads=1, dim=22, vdim=13, rot=6, mem_heads=1, mem_dim=20, mem_vdim=70, window=33, base=300.0),
    "layers that differ": dict(seed=5, kinds="apaapa", overrides={0: dict(v_mix=False, vdim=40, rot=16, ff=0), 1: dict(ff=30, window=1, kv_heads=4, rot=0), 3: dict(heads=2, dim=40, scale=0.3),
                                                                  4: dict(window=70, mem_heads=2, mem_dim=36, mem_vdim=8, cap=15.0), 5: dict(ff=0, heads=8, base=50.0)}),
    "no feed-forward": dict(seed=6, kinds="pa", ff=0, emb_scale=0.5),
}
_made, _refs = {}, {}


def model_of(name, dtype, **engine):
    """Configuration, weights and engine (models are built once per name and dtype, engines per call); page and slot order are shuffled."""
    if (name, dtype) not in _made:
        cfg, W = O.random_model(**MODELS[name])
        _made[name, dtype] = cfg, W, PufevikModel(PufevikConfig.from_dict(cfg), {k: torch.tensor(v) for k, v in W.items()}, "cuda", dtype)
    cfg, W, m = _made[name, dtype]
    engine.setdefault("max_tokens", 1024)
    eng = ServingEngine(m, **engine)
    rng = np.random.default_rng(0)
    rng.shuffle(eng.pool.free)
    if eng.states is not None:
        rng.shuffle(eng.states.free)
    return cfg, W, eng


def reference(name, cfg, W, tokens):
    key = (name, tuple(tokens))
    if key not in _refs:
        _refs[key] = O.forward(cfg, W, list(tokens))
    return _refs[key]


def prompt(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


LOGIT_TOL = {F32: 1e-4, BF16: 6e-2}


def close(got, want, dtype, spare=0):
    """f32: every position; bf16: all but a few. A head of the matrix memory whose query hardly meets what it holds has an output near zero, which its norm blows up
    together with the rounding in it: evaluating the reference on operands rounded to bf16 moves the same positions as far."""
    g, w = got.double().cpu().numpy(), np.asarray(want)
    assert g.shape == w.shape and np.isfinite(g).all()
    e = np.sqrt(((g - w) ** 2).mean(-1)) / np.sqrt((w ** 2).mean())
    over = int((e > LOGIT_TOL[dtype]).sum())
    assert over <= (0 if dtype == F32 else max(spare, len(e) // 12)), np.sort(e)[-5:]
    assert np.median(e) < LOGIT_TOL[dtype] / 2


def idle(eng):
    return eng.pool.num_free() == len(eng.pool.pages) and (eng.states is None or eng.states.num_free() == eng.max_sequences) and not eng._fed


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", MODELS)
def test_whole_prompts_and_residuals(name, dtype):
    cfg, W, eng = model_of(name, dtype)
    toks = prompt(cfg, 140, 1)
    taps, trace = [], []
    got = eng.step([StepEntry("a", toks, range(140))], ["a"], taps=taps)
    want = O.forward(cfg, W, toks, trace)
    close(got, want, dtype)
    for t, r in zip(taps, trace):
        close(t, r, dtype)
    assert len(taps) == len(cfg["layers"]) and "a" not in eng and idle(eng)
    close(eng.step([StepEntry("b", toks, [0, 17, 139])], ["b"]), want[[0, 17, 139]], dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", MODELS)
def test_token_by_token_equals_prefill(name, dtype):
    """From the very first token, over several page borders and past every window."""
    cfg, W, eng = model_of(name, dtype)
    assert eng.fast_decode == (dtype == BF16)
    toks = prompt(cfg, 90, 2)
    got = torch.cat([eng.step([StepEntry("a", [t], [0])]) for t in toks])
    close(got, reference(name, cfg, W, toks), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("size", [2, 7, 16, 33, 64])
def test_portions_of_prompts(size, dtype):
    cfg, W, eng = model_of("layers that differ", dtype)
    toks = prompt(cfg, 135, 3)
    out = []
    for i in range(0, 135, size):
        part = toks[i: i + size]
        out.append(eng.step([StepEntry("a", part, range(len(part)))]))
    close(torch.cat(out), reference("layers that differ", cfg, W, toks), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_batches_equal_each_request_alone_and_pages_and_slots_are_reused(dtype):
    """Unequal requests start together and decode together, shorter ones end earlier; further sets then run on the freed pages and slots."""
    cfg, W, eng = model_of("plain", dtype, max_tokens=400, max_sequences=4)
    for wave in range(3):
        lens = {f"{wave}a": (1, 20), f"{wave}b": (40, 3), f"{wave}c": (65, 12), f"{wave}d": (17, 17)}
        toks = {k: prompt(cfg, p + n, wave * 10 + p) for k, (p, n) in lens.items()}
        got = {k: [] for k in lens}

        def take(ids, logits):
            for i, k in enumerate(ids):
                got[k].append(logits[i])
        take(list(lens), eng.step([StepEntry(k, toks[k][:p], [p - 1]) for k, (p, _) in lens.items()]))
        with pytest.raises(InvalidArgument):
            eng.step([StepEntry("one more", [1])])
        for s in range(20):
            live = [k for k, (p, n) in lens.items() if s < n]
            take(live, eng.step([StepEntry(k, [toks[k][lens[k][0] + s]], [0]) for k in live], [k for k in live if s + 1 == lens[k][1]]))
        assert idle(eng)
        for k, (p, n) in lens.items():
            close(torch.stack(got[k]), reference("plain", cfg, W, toks[k])[p - 1: p + n], dtype)


def test_prompts_join_running_sequences_and_large_decode_batches():
    """One step that holds a prompt, a portion and single tokens; then twenty sequences decoding in one step."""
    cfg, W, eng = model_of("plain", BF16, max_tokens=1200)
    toks = {i: prompt(cfg, 30, 50 + i) for i in range(20)}
    eng.step([StepEntry(0, toks[0][:29]), StepEntry(1, toks[1][:10])])
    got = eng.step([StepEntry(0, toks[0][29:], [0]), StepEntry(1, toks[1][10:29], [18]), StepEntry(2, toks[2][:29], [0, 28])])
    want = [reference("plain", cfg, W, toks[0])[29], reference("plain", cfg, W, toks[1])[28], *reference("plain", cfg, W, toks[2])[[0, 28]]]
    close(got, np.stack(want), BF16)
    eng.release(0)
    eng.step([StepEntry(0, toks[0][:29])])
    eng.step([StepEntry(i, toks[i][:29]) for i in range(3, 20)])
    got = eng.step([StepEntry(i, [toks[i][29]], [0]) for i in range(20)])
    close(got, np.stack([reference("plain", cfg, W, toks[i])[29] for i in range(20)]), BF16)


def test_captured_decode_equals_plain_launches():
    """The run ahead of the capture leaves no trace in anybody's state."""
    cfg, W, a = model_of("layers that differ", BF16)
    _, _, b = model_of("layers that differ", BF16, use_graph=False)
    toks = prompt(cfg, 60, 6)
    for eng in (a, b):
        eng.step([StepEntry("s", toks[:5]), StepEntry("t", toks[:9])])
    for t in toks[5:30]:
        x, y = (e.step([StepEntry("s", [t], [0]), StepEntry("t", [t], [0])]) for e in (a, b))
        assert torch.equal(x, y)
    for t in toks[30:]:
        assert torch.equal(*(e.step([StepEntry("s", [t], [0])]) for e in (a, b)))
    close(a.step([StepEntry("s", [1], [0])]), reference("layers that differ", cfg, W, toks + [1])[-1:], BF16)


def test_long_prompts_and_long_decoding():
    """A prompt that walks in segments, then hundreds of decoded tokens over many pages."""
    cfg, W, eng = model_of("side by side only", BF16, max_tokens=1400)
    toks = prompt(cfg, 1300, 8)
    got = [eng.step([StepEntry("s", toks[:900], [0, 511, 512, 899])])] + [eng.step([StepEntry("s", [t], [0])]) for t in toks[900:]]
    want = reference("side by side only", cfg, W, toks)
    close(torch.cat(got), want[[0, 511, 512, 899, *range(900, 1300)]], BF16)


# -- generation --------------------------------------------------------------------------------------------------------------------------
def test_greedy_generation_through_the_scheduler():
    """f32 against the plain evaluation; bf16 decoding feeds its tokens back on the device and agrees with its own step-by-step run. More requests than
    fit at once, prompts cut into portions."""
    cfg, W, eng = model_of("plain", F32, max_tokens=160, max_sequences=3, prefill_chunk=11)
    prompts = [prompt(cfg, n, 70 + n) for n in (5, 30, 1, 17, 24)]
    out = eng.generate(prompts, GenerationConfig(max_new_tokens=7))
    assert out == [O.greedy(cfg, W, p, 7) for p in prompts] and idle(eng)
    stop = out[0][3]
    cut = eng.generate(prompts[:1], GenerationConfig(max_new_tokens=7, eos_token_id=stop))
    assert cut[0] == out[0][: out[0].index(stop) + 1]
    _, _, fast = model_of("plain", BF16, max_tokens=400)
    got = fast.generate(prompts, GenerationConfig(max_new_tokens=20))
    for p, o in zip(prompts, got):
        logits = fast.step([StepEntry("x", p, [len(p) - 1])])
        for t in o:
            top = torch.topk(logits[0], 2)
            assert t == int(top.indices[0]) or float(top.values[0] - logits[0, t]) < 0.05 * float(logits[0].std())
            logits = fast.step([StepEntry("x", [t], [0])])
        fast.release("x")
    assert idle(fast)
    fast.check()


def test_sequences_branch_and_step_back():
    """Forks copy the state; a sequence cut back to an earlier token continues as if the rest had never been fed (also after tokens fed back on the device)."""
    cfg, W, eng = model_of("plain", BF16)
    toks, other = prompt(cfg, 50, 12), prompt(cfg, 20, 13)
    eng.step([StepEntry("a", toks[:30])])
    eng.fork("a", "b")
    x = eng.step([StepEntry("a", toks[30:31], [0]), StepEntry("b", other[:1], [0])])
    close(x, np.stack([reference("plain", cfg, W, toks[:31])[-1], reference("plain", cfg, W, toks[:30] + other[:1])[-1]]), BF16)
    eng.decode_greedy(["a"], [5], 6)
    assert eng.length("a") == 37
    eng.truncate("a", 31)
    assert eng.length("a") == 31
    close(eng.step([StepEntry("a", toks[31:], range(19))]), reference("plain", cfg, W, toks)[31:], BF16)
    eng.truncate("a", 50)
    eng.truncate("b", 0)
    close(eng.step([StepEntry("b", other, range(20))]), reference("plain", cfg, W, other), BF16)
    kept = eng.decode_greedy(["b"], [7], 5)[0]
    eng.truncate("b", 23)
    close(eng.step([StepEntry("b", [3], [0])]), reference("plain", cfg, W, other + [7, *kept[:2], 3])[-1:], BF16)
    eng.release("a")
    eng.release("b")
    assert idle(eng)


def test_sampling_beam_and_speculative_decoding_over_the_engine():
    cfg, W, eng = model_of("plain", F32, max_tokens=900)
    p = prompt(cfg, 9, 90)
    want = O.greedy(cfg, W, p, 6)
    m = eng.as_cached_model()
    ids = torch.tensor([p], device="cuda")
    assert generate(m, m.new_cache, ids, GenerationConfig(max_new_tokens=6))[0, 9:].tolist() == want
    beam = beam_search(m, m.new_cache, ids, GenerationConfig(max_new_tokens=6, num_beams=3))

    def score(seq):
        lp = torch.log_softmax(torch.tensor(O.forward(cfg, W, seq[:-1])), -1)
        return float(sum(lp[i, seq[i + 1]] for i in range(8, len(seq) - 1)))
    assert score(beam[0].tolist()) >= score(p + want) - 1e-4
    _, _, other = model_of("plain", BF16, max_tokens=900)
    d = other.as_cached_model()                              # a draft that is not always right: rejected tokens are taken back
    spec, stats = speculative_generate(m, m.new_cache, d, d.new_cache, ids, SpecDecodeConfig(3, 6))
    assert spec[0, 9:].tolist() == want
    c = GenerationConfig(max_new_tokens=5, seed=3).with_temperature(0.9).with_top_k(8)
    one, two = eng.generate([p, p[:4]], c), eng.generate([p], c)
    assert one[0] == two[0] and len(one[1]) == 5                          # a request's draws do not depend on its batch
    import gc
    gc.collect()
    assert idle(eng) and idle(other)


def test_trace_replay_program(tmp_path):
    from ferrotorch_b200.serialize import save_safetensors
    cfg, W = O.random_model(**MODELS["odd sizes"])
    d, out = tmp_path / "model", tmp_path / "out"
    d.mkdir()
    out.mkdir()
    (d / "config.json").write_text(json.dumps(cfg))
    save_safetensors({k: torch.tensor(v).to(BF16) for k, v in W.items()}, d / "model.safetensors")
    toks = prompt(cfg, 20, 4)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:12], "want": [3, 11]}, {"id": "b", "tokens": toks[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[12:13], "want": []}, {"id": "b", "tokens": toks[1:2], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[13:14], "want": [0]}], "end": ["a"]}]
    exe = Path(__file__).resolve().parents[1] / "bin" / "trace_run"
    r = subprocess.run([sys.executable, str(exe), "--model", str(d), "--dtype", "float32", "--out", str(out), "--max-tokens", "32"],
                       input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = O.forward(cfg, W, toks)
    for n, rows in ((0, [3, 11]), (2, [13])):
        close(torch.tensor(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])), want[rows], F32)
    assert not (out / "1.f32").exists()


def test_random_weights_and_refused_models():
    cfg = PufevikConfig.pattern("pa", 64, 32, 24, 4, 2, 16, 16, 8, 2, 16, 16)
    W = RandomPufevikWeights(cfg)
    assert set(W.keys()) == set(cfg.tensor_shapes()) and W["l1.mix.vmix"].shape == ()
    eng = ServingEngine(PufevikModel(cfg, W), max_tokens=32, max_sequences=2)
    assert len(eng.generate([[1, 2, 3]], GenerationConfig(max_new_tokens=4))[0]) == 4 and idle(eng)
    PufevikModel(cfg, {k: W[k] for k in W.keys() if k != "l1.mix.vmix"})            # the first mixing layer's own weight is not read
    with pytest.raises(InvalidArgument):
        PufevikModel(cfg, {k: W[k] for k in W.keys() if k != "l0.mix.right.i.b"})
    with pytest.raises(InvalidArgument):
        PufevikModel(cfg, W, dtype=torch.float16)
