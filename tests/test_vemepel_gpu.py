"""Vemepel on the device against the plain f64 evaluation in ``vemepel_oracle``: every mechanism by itself, then prompts, portions of prompts, decoding, batches, reuse of pages and
state slots, and generation."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import vemepel_oracle as O
from ferrotorch_b200 import _lib
from ferrotorch_b200.errors import InvalidArgument
from ferrotorch_b200.models import (DecodeState, ExpertConfig, GenerationConfig, MoeConfig, RandomVemepelWeights, RowBatch, ServingEngine, SpecDecodeConfig, StepEntry, VemepelConfig, VemepelModel,
                                    beam_search, generate, load_engine, speculative_generate)
from ferrotorch_b200.nn import PagedRowCache, PagePool, StateSlots
from ferrotorch_b200.ops import (DensePolyWeights, ExpertStack, GqaDecodeBuffers, GqaDims, GqaWeights, LatentDecodeBuffers, LatentDims, LatentWeights, MoeRouting, MoeSmallBuffers, MoeWeights,
                                 RouteRule, SublayerOutput, TokenShift, dense_poly_rows, depth_embed, depth_update, gqa_attention_decode, gqa_attention_rows, latent_attention_decode,
                                 latent_attention_rows, moe_rows, moe_small, pack_head_columns, poly_norm_planes, poly_norm_rows, token_shift)
from ferrotorch_b200.ops.gqa_attention import GATE_ELEMENT, GATE_HEAD
from ferrotorch_b200.ops.latent_attention import rotary_pair_tables
from ferrotorch_b200.ops.streams import padded_vector, round_up

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
GPU = torch.device("cuda")


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


class Pages:
    """A page cache full of other sequences' leftovers, with shuffled pages (and slots)."""

    def __init__(self, row, dtype, rng, tokens=2048, states=None):
        self.pool = PagePool(tokens // 16 + 8, 16)
        rng.shuffle(self.pool.free)
        self.cache = PagedRowCache(self.pool, [row], "cuda", dtype, states)
        self.cache.rows[0].normal_()
        self.blocks = tokens // 16

    def open(self, ids):
        for s in ids:
            self.cache.add_sequence(s)

    def batch(self, parts):
        entries = [StepEntry(s, [0] * (hi - lo)) for s, (_, lo, hi) in parts.items()]
        for e in entries:
            self.cache.reserve(e.id, self.cache.lengths[e.id] + len(e.tokens))
        return RowBatch(entries, self.cache, GPU, self.blocks)

    def advance(self, parts):
        for s, (_, lo, hi) in parts.items():
            self.cache.lengths[s] += hi - lo

    def state(self, ids):
        st = DecodeState("cuda", self.blocks)
        for s in ids:
            self.cache.reserve(s, self.cache.lengths[s] + 1)
        slots = None if self.cache.states is None else [self.cache.states.slot[s] for s in ids]
        st.load([0] * len(ids), [self.cache.lengths[s] for s in ids], self.cache.block_table(ids, self.blocks), slots)
        return st


def in_portions(step, P, cuts):
    """Runs ``step`` over the ragged portions between ``cuts``; output rows by sequence."""
    got = {s: [] for s in P}
    for i in range(len(next(iter(cuts.values()))) - 1):
        parts = {s: (P[s], c[i], c[i + 1]) for s, c in cuts.items() if c[i + 1] > c[i]}
        out, at = step(parts), 0
        for s, (_, lo, hi) in parts.items():
            got[s].append(out[at: at + hi - lo])
            at += hi - lo
    return {s: torch.cat(g) for s, g in got.items()}


# -- token shift and averages over depth ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [4, 7, 260, 2052, 9001])
def test_token_shift_of_ragged_portions(dtype, width):
    """Portions of one, two and many tokens of several sequences; a slot that is used again; a sequence that starts in a slot full of leftovers."""
    rng = np.random.default_rng(width)
    share, w, eps = rounded(rng.uniform(-0.3, 1.2, width), F32), rounded(rng.standard_normal(width), F32), 1e-3
    states = StateSlots(3, [round_up(width, 4)], "cuda")
    states.data[0].fill_(float("nan"))
    P = Pages(0, dtype, rng, 512, states)
    shift = TokenShift(padded_vector(dev(share), "cuda"), states.data[0])
    wp, ld = padded_vector(dev(w), "cuda"), round_up(width, 8)
    tol = 2e-6 if dtype == F32 else 6e-3

    def step(parts):
        b = P.batch(parts)
        x = padded(np.concatenate([p[lo:hi] for p, lo, hi in parts.values()]), F32)
        rstd = 1.0 / torch.sqrt(x.double().pow(2).mean(-1) + eps).float()
        h = torch.full((x.shape[0], ld), float("nan"), device="cuda", dtype=dtype)[:, :width]
        token_shift(x, rstd, wp, shift, b.memory_plan(0).spans, b.seq_of, h, x.shape[0], width)
        P.advance(parts)
        return h
    for wave in range(2):
        X = {s: rounded(rng.standard_normal((n, width)) + 0.5, F32) for s, n in (("a", 40), ("b", 1), ("c", 33))}
        P.open(X)
        got = in_portions(step, X, {"a": [0, 2, 3, 12, 40], "b": [0, 1, 1, 1, 1], "c": [0, 7, 9, 10, 33]})
        for s in X:
            n = O.rms(X[s], eps) * w
            assert rel(got[s], O.token_shift(n, share)) < tol
            assert np.abs(states.data[0][states.slot[s], :width].double().cpu().numpy() - n[-1]).max() < 1e-5 * np.abs(n).max()
            P.cache.free_sequence(s)
    assert states.num_free() == 3


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width", [(1, 5), (3, 2052), (16, 640), (300, 68), (2, 9001), (7, 30000)])
def test_residual_with_norms_behind_sublayers_and_averages_over_depth(dtype, rows, width):
    rng = np.random.default_rng(rows)
    table, ids, ld, eps = rounded(rng.standard_normal((11, width)), dtype), rng.integers(0, 11, rows), round_up(width, 8), 1e-3
    streams = torch.full((6, rows, ld), float("nan"), device="cuda")
    x, results = streams[0], streams[1:]
    h, rstd = torch.full((rows, ld), float("nan"), device="cuda", dtype=dtype)[:, :width], torch.full((rows,), float("nan"), device="cuda")
    w_out, w_next = rounded(rng.standard_normal((2, width)), F32)
    po, pn = padded_vector(dev(w_out), "cuda"), padded_vector(dev(w_next), "cuda")
    tol = 1e-5 if dtype == F32 else 1e-2
    idt, tab = torch.as_tensor(ids).cuda(), padded(table, dtype)
    depth_embed(idt, tab, x, results, pn, eps, rows, h)
    want = [table[ids]]
    assert torch.equal(x[:, :width], results[0, :, :width]) and rel(x[:, :width], want[0]) < 1e-6 and rel(h, O.rms(want[0], eps) * w_next) < tol
    depth_embed(idt, tab, x, results, None, eps, rows, rstd=rstd)
    assert rel(rstd[:, None], 1.0 / np.sqrt((want[0] ** 2).mean(-1, keepdims=True) + eps)) < 1e-6
    expert_rows = rounded(rng.standard_normal((3 * rows + 2, width)), dtype)
    row_of = rng.permutation(3 * rows + 2)[: 3 * rows].reshape(rows, 3)
    experts = dict(rows=padded(expert_rows, dtype), row_of=torch.as_tensor(row_of, dtype=torch.int32).cuda().contiguous(), top=3)
    old = want[0]
    for n, form in enumerate(("planes", "experts", "both", "planes"), 1):
        p = split_planes(rng.standard_normal((rows, width)), 5, rng, pad=rows + 1)
        y = (p[:, :rows, :width].double().sum(0).cpu().numpy() if form != "experts" else 0.0) + (expert_rows[row_of].sum(1) if form != "planes" else 0.0)
        out = SublayerOutput(planes=p if form != "experts" else None, **(experts if form != "planes" else {}))
        avg = rounded(rng.standard_normal(n + 1), F32)
        last = n == 4
        before = x.clone()
        rstd.fill_(7.0)
        h.fill_(7.0)
        depth_update(x, results, dev(avg), out, po, pn if last else None, eps, dtype, rows, width, h=h if last else None, rstd=None if last else rstd, store=not last)
        want.append(old + O.rms(y, eps) * w_out)
        new = O.depth_average(want, avg)
        if last:
            assert rel(h, O.rms(new, eps) * w_next) < tol and torch.equal(x[:, :width], before[:, :width]) and bool((rstd == 7.0).all())
        else:
            assert rel(results[n, :, :width], want[n]) < 5e-6 and rel(x[:, :width], new) < 5e-6 and bool((h == 7.0).all())
            assert rel(rstd[:, None], 1.0 / np.sqrt((new ** 2).mean(-1, keepdims=True) + eps)) < 1e-5
            want[n], old = results[n, :, :width].double().cpu().numpy(), x[:, :width].double().cpu().numpy()
    # one token per sequence, its state in a slot
    if rows <= 16:
        share = rounded(rng.uniform(0, 1, width), F32)
        data = dev(rng.standard_normal((rows + 2, round_up(width, 4))))
        slots = torch.as_tensor(rng.permutation(rows + 2)[:rows], dtype=torch.int32).cuda()
        positions = torch.as_tensor([0 if r % 3 == 1 else 5 for r in range(rows)], dtype=torch.int32).cuda()
        kept = data.clone()
        prev = data[slots.long(), :width].double().cpu().numpy() * (positions.cpu().numpy() > 0)[:, None]
        depth_embed(idt, tab, x, results, pn, eps, rows, h, shift=TokenShift(padded_vector(dev(share), "cuda"), data), slots=slots, positions=positions)
        norm = O.rms(table[ids], eps) * w_next
        assert rel(h, (1 - share) * norm + share * prev) < tol and rel(data[slots.long(), :width], norm) < 1e-5
        spare = [s for s in range(rows + 2) if s not in slots.tolist()]
        assert torch.equal(data[spare], kept[spare])
        p = split_planes(rng.standard_normal((rows, width)), 3, rng, pad=rows)
        avg = rounded([0.4, 1.1], F32)
        positions[:] = 6
        depth_update(x, results, dev(avg), SublayerOutput(planes=p), po, pn, eps, dtype, rows, width, h, shift=TokenShift(padded_vector(dev(share), "cuda"), data), slots=slots, positions=positions)
        prev, new = norm, O.rms(0.4 * table[ids] + 1.1 * (table[ids] + O.rms(p[:, :rows, :width].double().sum(0).cpu().numpy(), eps) * w_out), eps) * w_next
        assert rel(h, (1 - share) * new + share * prev) < tol and rel(data[slots.long(), :width], new) < 1e-5


# -- dense feed-forward ----------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width,ff", [(24, 8), (40, 33), (64, 700), (16, 2050), (8, 9001), (8, 16390)])
def test_dense_feed_forward_of_normed_powers(dtype, width, ff):
    rng = np.random.default_rng(ff)
    act = rounded([0.7, -0.4, 1.3, 0.25], F32)
    W = {k: rounded(rng.standard_normal(s) / s[-1] ** 0.5 * 1.5, dtype) for k, s in (("up", (ff, width)), ("down", (width, ff)))}
    W["act"] = act
    eps = 1e-2
    w = DensePolyWeights.pack(torch.tensor(W["up"]), torch.tensor(W["down"]), torch.tensor(act), eps, "cuda", dtype)
    for rows in (1, 5, 130, 150):
        h = rounded(2.0 * rng.standard_normal((rows, width)), dtype)
        assert rel(dense_poly_rows(padded(h, dtype), w).planes[0], O.dense(h, W, eps)) < (1e-5 if dtype == F32 else 3e-2)
        z = rounded(np.exp(rng.standard_normal((rows, 1))) * rng.standard_normal((rows, ff)), dtype)
        assert rel(poly_norm_rows(padded(z, dtype), w.coef, eps), O.poly_norm(z, act, eps)) < (1e-5 if dtype == F32 else 6e-3)
    z = rounded(2.0 * rng.standard_normal((7, ff)), F32)
    out = torch.zeros(16, round_up(ff, 8), device="cuda", dtype=BF16)[:, :ff]
    poly_norm_planes(split_planes(z, 3, rng), 3, 7, w.coef, eps, out)
    assert rel(out[:7], O.poly_norm(z, act, eps)) < 6e-3 and not out[7:].any()


# -- differential attention within chunks ----------------------------------------------------------------------------------------------------
class DifferentialRig(Pages):
    """A layer with keys and values of its own and one that reads them (with queries, chunks, scale and heads of its own), fed with projection rows."""

    def __init__(self, D, dtype, seed=0, blend=0.45, second=None):
        self.dtype, self.rng, self.blend = dtype, np.random.default_rng(seed), blend
        s = dict(heads=D.heads, scale=D.scale * 0.8, chunk=D.chunk + 5 if D.chunk else 9, diff=0.1)
        s.update(second or {})
        self.D = [D, GqaDims(s["heads"], D.kv_heads, D.dim, D.vdim, 0, s["scale"], D.eps, norm=False, chunk=s["chunk"], maps=2, diff=s["diff"], own=False)]
        self.w = [GqaWeights.pack(d, None, None, "cuda", blend=b) for d, b in zip(self.D, (blend, -0.3))]
        super().__init__(D.row, dtype, self.rng)

    def projections(self, n):
        D = self.D[0]
        out = {k: rounded(self.rng.standard_normal((n, *s)), self.dtype) for k, s in (("k", (D.kv_heads, 2, D.dim)), ("v", (D.kv_heads, D.vdim)))}
        out["q"] = [rounded(self.rng.standard_normal((n, d.heads, 2, d.dim)), self.dtype) for d in self.D]
        return out

    def rows(self, P, i, lo, hi):
        D = self.D[i]
        parts = [(P["q"][i], 2 * D.heads, D.dim)] + ([(P["k"], 2 * D.kv_heads, D.dim), (P["v"], D.kv_heads, D.vdim)] if D.own else [])
        return torch.cat([pack_head_columns(torch.tensor(t[lo:hi]).flatten(1), n, s, "cuda", self.dtype) for t, n, s in parts], 1).contiguous()

    def reference(self, P):
        n = P["k"].shape[0]
        out = [O.differential(P["q"][i], P["k"], P["v"], D.scale, O.visible(n, D.chunk or None), w.blend, D.diff, D.eps) for i, (D, w) in enumerate(zip(self.D, self.w))]
        return np.concatenate([o.reshape(n, -1) for o in out], 1)

    def heads_of(self, out, D):
        return out.view(out.shape[0], D.heads, D.v16)[..., : D.vdim].flatten(1)

    def step(self, parts):
        batch, got = self.batch(parts), []
        for i, D in enumerate(self.D):
            x = torch.cat([self.rows(p, i, lo, hi) for p, lo, hi in parts.values()])
            out = torch.full((x.shape[0], D.out_cols), float("nan"), device="cuda", dtype=self.dtype)
            gqa_attention_rows(x, self.w[i], batch, self.cache.rows[0], None, None, None, out)
            got.append(self.heads_of(out, D))
        self.advance(parts)
        return torch.cat(got, 1)

    def decode(self, parts, splits=None):
        """One token per sequence: {sequence: (projections, token)}."""
        B, ids, got = len(parts), list(parts), []
        state = self.state(ids)
        for i, D in enumerate(self.D):
            planes = split_planes(torch.cat([self.rows(p, i, t, t + 1) for p, t in parts.values()]).double().cpu().numpy(), 3, self.rng)
            b = GqaDecodeBuffers(D, 16, self.blocks * 16, "cuda", splits)
            out = torch.zeros(16, D.out_cols, device="cuda", dtype=BF16)
            for _ in range(2):                              # the second run finds the counters as the first one left them
                gqa_attention_decode(planes, 3, self.w[i], b, state, self.cache.rows[0], None, None, B, 0, out)
            assert not b.counters.any() and not out[B:].any()
            got.append(self.heads_of(out, D)[:B])
        for s in ids:
            self.cache.lengths[s] += 1
        return torch.cat(got, 1)


def dims(heads, kv_heads, dim, vdim, chunk=0, diff=0.6):
    return GqaDims(heads, kv_heads, dim, vdim, 0, 1.3 * dim ** -0.5, 1e-4, norm=False, chunk=chunk, maps=2, diff=diff)


DIFFERENTIAL = {
    "one head": (dims(1, 1, 8, 8), None),
    "groups": (dims(8, 2, 48, 40, 30), None),
    "a chunk of one": (dims(4, 2, 32, 16, 1, 0.0), None),
    "odd sizes": (dims(5, 1, 23, 11, 7), dict(heads=3)),
    "chunks of a block": (dims(4, 1, 64, 64, 64), dict(chunk=128)),
    "wide values": (dims(2, 2, 64, 128, 100), dict(chunk=0)),
    "widest joined": (dims(4, 4, 128, 128, 130), dict(heads=8)),
    "values beyond the joined kernel": (dims(4, 2, 40, 200, 48), None),
    "keys beyond the joined kernel": (dims(2, 1, 160, 100, 70), None),
    "beyond the tiled kernel": (dims(2, 1, 40, 300, 70), None),
    "more rows than a tile": (dims(20, 1, 16, 24, 33), dict(heads=40)),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", DIFFERENTIAL)
def test_differential_attention_of_ragged_prompts_and_portions(case, dtype):
    D, second = DIFFERENTIAL[case]
    rig = DifferentialRig(D, dtype, 1, second=second)
    P = {s: rig.projections(n) for s, n in (("a", 150), ("b", 1), ("c", 293))}
    rig.open(P)
    got = in_portions(rig.step, P, {"a": [0, 2, 71, 150], "b": [0, 1, 1, 1], "c": [0, 129, 131, 293]})
    for s in P:
        assert rel(got[s], rig.reference(P[s])) < (2e-5 if dtype == F32 else 3e-2), s


@pytest.mark.parametrize("splits", [None, 1, 7])
@pytest.mark.parametrize("case", DIFFERENTIAL)
def test_differential_decode_matches_the_whole_sequence(case, splits):
    D, second = DIFFERENTIAL[case]
    assert D.decode_supported()
    rig = DifferentialRig(D, BF16, 2, second=second)
    lens = {"a": 0, "b": 15, "c": 16, "d": 200, "e": 64}
    P = {s: rig.projections(n + 3) for s, n in lens.items()}
    want = {s: rig.reference(p) for s, p in P.items()}
    rig.open(P)
    rig.step({s: (P[s], 0, n) for s, n in lens.items() if n})
    for t in range(3):
        got = rig.decode({s: (P[s], n + t) for s, n in lens.items()}, splits)
        assert rel(got, np.stack([want[s][n + t] for s, n in lens.items()])) < 3e-2


@pytest.mark.parametrize("heads,kv_heads,chunk", [(4, 1, 16), (6, 2, 37), (8, 1, 64), (3, 3, 100), (4, 2, 129), (2, 1, 0)])
@pytest.mark.parametrize("target", [0, 15, 63, 64, 74, 130])
@pytest.mark.parametrize("map_", [0, 1])
def test_one_key_stands_out_inside_its_chunk(heads, kv_heads, chunk, target, map_):
    """One key of one map meets every query with a score far above all others; the other map weighs all it sees alike. In prompts, portions and decoding, around page, block
    and chunk borders, also in the layer that reads these keys with chunks of its own."""
    rig = DifferentialRig(GqaDims(heads, kv_heads, 32, 16, 0, 0.6, 1e-6, norm=False, chunk=chunk, maps=2, diff=0.2), BF16, target, blend=0.5)
    n = 270
    P = rig.projections(n)
    for q in P["q"]:
        q[:, :, map_] = 0.0
        q[:, :, map_, 31] = 8.0
        q[:, :, 1 - map_] = 0.0
    P["k"][:, :, map_, 31] = 0.0
    P["k"][target, :, map_] = 0.0
    P["k"][target, :, map_, 31] = 6.0
    want = rig.reference(P)
    first, last = (target // chunk * chunk, (target // chunk + 1) * chunk) if chunk else (0, n)
    mean = lambda i: np.repeat(P["v"][(i // chunk * chunk if chunk else 0): i + 1].mean(0), heads // kv_heads, 0)
    for i in range(first, min(last, n)):                     # the first layer's outputs by hand
        if i >= target:
            v = np.repeat(P["v"][target], heads // kv_heads, 0)
            o = v - 0.5 * mean(i) if map_ == 0 else mean(i) - 0.5 * v
            assert np.abs(want[i, : heads * 16] - (O.rms(o, 1e-6) * 0.8).reshape(-1)).max() < 1e-3
    rig.open(["whole", "parts", "steps"])
    assert rel(rig.step({"whole": (P, 0, n)}), want) < 2e-2
    got = [rig.step({"parts": (P, lo, hi)}) for lo, hi in ((0, 66), (66, 68), (68, 200), (200, n))]
    assert rel(torch.cat(got), want) < 2e-2
    lo, hi = max(0, min(last, n) - 3), min(n, last + 4)
    rig.step({"steps": (P, 0, lo)})
    for t in range(lo, hi):
        assert rel(rig.decode({"steps": (P, t)}), want[t].reshape(1, -1)) < 2e-2, t


# -- gated latent attention ------------------------------------------------------------------------------------------------------------------
# heads, dim, rotated, vdim, latent
LATENT = {"small": (3, 16, 0, 20, 32), "small, rotated": (3, 16, 8, 20, 32), "odd sizes": (5, 23, 0, 11, 33), "odd sizes, rotated": (5, 23, 6, 11, 33), "one of each": (1, 8, 2, 1, 1), "no rotation, one value": (2, 8, 0, 1, 8),
          "wide": (2, 128, 64, 128, 64), "wide, no rotation": (2, 128, 0, 128, 200), "many heads": (34, 32, 16, 16, 48), "beyond the tiled kernel": (2, 300, 8, 24, 16), "gates beyond the tiled kernel": (2, 300, 0, 24, 16),
          "large latent": (2, 40, 20, 40, 530)}


class LatentRig(Pages):
    def __init__(self, sizes, dtype, seed=0, width=40, base=700.0):
        H, d, e, dv, r = sizes
        self.dtype, self.rng, self.eps, self.width = dtype, np.random.default_rng(seed), 1e-4, width
        self.m = dict(heads=H, dim=d, vdim=dv, kv_rank=r, scale=1.2 * (d + e) ** -0.5)
        if e:
            self.m.update(rot_dim=e, rot=dict(base=base, dims=e))

        def mat(o, i, s=1.0):
            return rounded(self.rng.standard_normal((o, i)) * s / i ** 0.5, dtype)
        self.W = {"q": mat(H * (d + e), width, 1.5), "dkv": mat(r + e, width), "dkv.norm": rounded(1 + 0.2 * self.rng.standard_normal(r), F32), "uk": mat(H * d, r, 1.5), "uv": mat(H * dv, r),
                  "g": mat(H * dv if e else H, width, 2.0), "o": mat(width, H * dv)}
        self.D = LatentDims(H, d, e, dv, r, self.m["scale"], self.eps, gate=GATE_ELEMENT if e else GATE_HEAD)
        self.tables = rotary_pair_tables(1024, e, base, "cuda") if e else (None, None)
        self.pack()
        super().__init__(self.D.row, dtype, self.rng, 1024)

    def pack(self):
        t = {k: torch.tensor(v) for k, v in self.W.items()}
        self.w = LatentWeights.pack(self.D, *(t[k] for k in ("q", "dkv", "dkv.norm", "uk", "uv", "o")), "cuda", self.dtype, gate=t["g"])

    def inputs(self, n):
        return rounded(self.rng.standard_normal((n, self.width)), self.dtype)

    def reference(self, P):
        return O.latent_mixer(P, self.W, self.m, self.eps)

    def step(self, parts):
        batch = self.batch(parts)
        out = latent_attention_rows(padded(np.concatenate([p[lo:hi] for p, lo, hi in parts.values()]), self.dtype), self.w, batch, self.cache.rows[0], *self.tables).planes[0]
        self.advance(parts)
        return out

    def decode(self, parts):
        B, ids = len(parts), list(parts)
        state = self.state(ids)
        h = np.concatenate([p[t: t + 1] for p, t in parts.values()])
        b = LatentDecodeBuffers(self.D, 16, self.blocks * 16, "cuda")
        planes = split_planes(h @ self.w.proj.double().cpu().numpy().T, 3, self.rng)
        a = latent_attention_decode(planes, 3, self.w, b, state, self.cache.rows[0], *self.tables, B)
        for s in ids:
            self.cache.lengths[s] += 1
        return a[:B].double() @ self.w.out.double().t()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", LATENT)
def test_latent_attention_of_prompts_and_portions(case, dtype):
    rig = LatentRig(LATENT[case], dtype, 1)
    P = {s: rig.inputs(n) for s, n in (("a", 150), ("b", 1), ("c", 203))}
    rig.open(P)
    got = in_portions(rig.step, P, {"a": [0, 2, 71, 150], "b": [0, 1, 1, 1], "c": [0, 129, 131, 203]})
    for s in P:
        assert rel(got[s], rig.reference(P[s])) < (2e-5 if dtype == F32 else 3e-2), s


@pytest.mark.parametrize("case", [c for c in LATENT if "beyond" not in c])
def test_latent_decode_matches_the_whole_sequence(case):
    rig = LatentRig(LATENT[case], BF16, 2)
    assert rig.D.decode_supported()
    lens = {"a": 0, "b": 15, "c": 16, "d": 200, "e": 64}
    P = {s: rig.inputs(n + 3) for s, n in lens.items()}
    want = {s: rig.reference(p) for s, p in P.items()}
    rig.open(P)
    rig.step({s: (P[s], 0, n) for s, n in lens.items() if n})
    for t in range(3):
        got = rig.decode({s: (P[s], n + t) for s, n in lens.items()})
        assert rel(got, np.stack([want[s][n + t] for s, n in lens.items()])) < 4e-2


@pytest.mark.parametrize("target", [0, 15, 16, 63, 64, 130])
@pytest.mark.parametrize("case", ["small", "small, rotated"])
def test_one_latent_stands_out_however_far_back(target, case):
    """The input of one token meets every later query with a score far above all others."""
    rig = LatentRig(LATENT[case], BF16, target)
    m, n, W = rig.m, 210, rig.W
    H, d, e = m["heads"], m["dim"], m.get("rot_dim", 0)
    P = rig.inputs(n)
    q = rounded(rig.rng.standard_normal(d), BF16)
    W["q"][:] = 0.0                                          # queries are one vector without a rotated part, whatever the input; keys of one latent direction point along it
    W["q"].reshape(H, d + e, -1)[:, :d, 0] = 3.0 * q
    W["uk"][:] = 0.0
    W["uk"][:, 3] = np.tile(q, H)
    W["dkv"][3] = 0.0
    W["dkv"][3, 1] = 1.0
    rig.pack()
    P[:, 0] = 1.0
    P[:, 1] = 0.0
    P[target, 1] = 30.0
    want = rig.reference(P)
    c, _ = O.latent_of(P, W, m, rig.eps)
    g = O.sigmoid(P[-1] @ W["g"].T).reshape(H, -1)
    alone = ((c[target] @ W["uv"].T).reshape(H, -1) * g).reshape(-1) @ W["o"].T
    assert np.abs(want[-1] - alone).max() < 0.05 * np.abs(alone).max()
    rig.open(["whole", "parts", "steps"])
    assert rel(rig.step({"whole": (P, 0, n)}), want) < 3e-2
    assert rel(torch.cat([rig.step({"parts": (P, lo, hi)}) for lo, hi in ((0, 66), (66, 68), (68, n))]), want) < 3e-2
    rig.step({"steps": (P, 0, target + 1)})
    for t in range(target + 1, target + 5):
        assert rel(rig.decode({"steps": (P, t)}), want[t: t + 1]) < 4e-2


# -- mixture of experts ----------------------------------------------------------------------------------------------------------------------
def make_moe(dtype, width, experts, top, ff, seed=0):
    rng = np.random.default_rng(seed)
    W = {"router": rounded(rng.standard_normal((experts, width)) * 2 / width ** 0.5, dtype), "router.b": rounded(0.8 * rng.standard_normal(experts), F32)}
    for i in range(experts):
        W.update({f"e{i}.{k}": rounded(rng.standard_normal(s) * 1.5 / s[1] ** 0.5, dtype) for k, s in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))})
    stack = ExpertStack.pack(*([torch.tensor(W[f"e{i}.{k}"]) for i in range(experts)] for k in ("gate", "up", "down")), float("inf"), "cuda", dtype)
    w = MoeWeights(padded(W["router"], dtype), stack, None, width, top, form="silu", rule=RouteRule(padded_vector(torch.tensor(W["router.b"]), "cuda"), softmax=True))
    return W, dict(router=dict(top=top)), w


def clear_rows(W, top, rng, n, dtype):
    """Token rows whose choice of experts is not a close call."""
    rows = []
    while len(rows) < n:
        h = rounded(rng.standard_normal((1, W["router"].shape[1])), dtype)[0]
        z = np.sort(W["router"] @ h + W["router.b"])[::-1]
        if top == len(z) or z[top - 1] - z[top] > 0.05:
            rows.append(h)
    return np.stack(rows)


MIXTURES = [(40, 8, 3, 24), (56, 12, 4, 33), (64, 9, 2, 8), (32, 6, 1, 40), (48, 64, 6, 16), (24, 4, 4, 16), (20, 1, 1, 16)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", MIXTURES)
def test_mixture_of_any_number_of_tokens(dtype, case):
    W, mlp, w = make_moe(dtype, *case)
    rng = np.random.default_rng(1)
    for n in (1, 17, 300):
        h = clear_rows(W, case[2], rng, n, dtype)
        y = moe_rows(padded(h, dtype), w)
        assert y.planes is None
        assert rel(y.rows.double()[y.row_of.view(-1, y.top).long()].sum(1)[:, : case[0]], O.mixture(h, W, mlp)) < (1e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("case", MIXTURES)
def test_mixture_of_a_decode_step(case):
    W, mlp, w = make_moe(BF16, *case)
    rng = np.random.default_rng(2)
    b = MoeSmallBuffers.allocate([w], "cuda")
    b.planes.fill_(float("nan"))
    for n in (1, 2, 8, 9, 16):
        h = clear_rows(W, case[2], rng, n, BF16)
        buf = torch.zeros(16, round_up(case[0], 8), device="cuda", dtype=BF16)[:, : case[0]]
        buf[:n] = dev(h, BF16)
        y = moe_small(buf, w, b, n)
        assert rel(y.planes[: y.count, :n, : case[0]].double().sum(0), O.mixture(h, W, mlp)) < 2e-2


def route_on_device(z, bias, top):
    """Choice and weights of both routers for given logits: the router's weights are the logits, the tokens unit vectors."""
    T, E = z.shape
    zb = rounded(z, BF16)
    router = torch.zeros(E, 16, device="cuda", dtype=BF16)
    router[:, :T] = dev(zb.T, BF16)
    h = torch.zeros(16, 16, device="cuda", dtype=BF16)
    h[range(T), range(T)] = 1.0
    stack = ExpertStack.pack([torch.zeros(8, 16)] * E, [torch.zeros(8, 16)] * E, [torch.zeros(16, 8)] * E, float("inf"), "cuda", BF16)
    w = MoeWeights(router, stack, None, 16, top, form="silu", rule=RouteRule(dev(bias), softmax=True))
    r = MoeRouting.choose(h[:T], w)
    many = (r.expert.view(T, top).cpu().numpy(), r.score.view(T, top).cpu().numpy())
    b = MoeSmallBuffers.allocate([w], "cuda")
    moe_small(h, w, b, T)
    chosen = np.full((T, top), -1)
    for a in range(int(b.n_active)):
        for t in range(T):
            p = int(b.pair_of.view(-1, 16)[a, t])
            if p >= 0:
                chosen[t, p % top] = int(b.ids[a])
    return zb, many, (chosen, b.score[: T * top].view(T, top).cpu().numpy())


@pytest.mark.parametrize("experts,top,spread", [(8, 3, 3.0), (5, 1, 3.0), (6, 6, 3.0), (200, 20, 10.0), (12, 4, 60.0)])
def test_routing_goes_by_biased_logits_with_softmax_weights(experts, top, spread):
    rng = np.random.default_rng(experts + top)
    z, bias = spread * rng.standard_normal((16, experts)), spread * rng.standard_normal(experts)
    zb, many, few = route_on_device(z, bias, top)
    for t in range(16):
        e, w = O.route(zb[t] + np.float32(bias).astype(np.float64), top)
        for got_e, got_w in (many, few):
            assert got_e[t].tolist() == list(e) and np.abs(got_w[t] - w).max() < 1e-5


# -- the model ---------------------------------------------------------------------------------------------------------------------------
MODELS = {
    "plain": dict(seed=1, kinds="arl"),
    "shared keys": dict(seed=2, kinds="araala", overrides={2: dict(kv_from=0), 3: dict(kv_from=0, chunk=50, diff=0.1, heads=6, scale=0.2), 5: dict(chunk=7)}),
    "odd sizes": dict(seed=3, kinds="rala", vocab=101, width=53, ff=37, dense_ff=35, heads=5, kv_heads=1, dim=11, vdim=13, chunk=33, rot=6, base=300.0, lat_heads=2, lat_dim=21, lat_vdim=9, kv_rank=19,
                      experts=6, top=2, logit_scale=1.9, eps=1e-3),
    "layers that differ": dict(seed=4, kinds="larar", overrides={0: dict(mlp="dense", lat_heads=7), 1: dict(chunk=1, mlp=None, diff=0.8), 2: dict(experts=5, top=4, rot=20, base=50.0, kv_rank=8),
                                                                 3: dict(chunk=0, kv_heads=4, dim=40, vdim=150, mlp="dense", dense_ff=9), 4: dict(mlp=None, lat_vdim=8, scale=0.3)}),
    "dense": dict(seed=5, kinds="ala", mlp="dense", chunk=16, heads=2, kv_heads=2, overrides={2: dict(kv_from=0)}),
    "no feed-forward": dict(seed=6, kinds="rl", mlp=None, logit_scale=0.25),
    "one layer": dict(seed=7, kinds="a", heads=1, kv_heads=1, experts=4, top=1),
}
_made, _refs = {}, {}


def model_of(name, dtype, **engine):
    """Configuration, weights and engine (models are built once per name and dtype, engines per call); page and slot order are shuffled, slots are full of leftovers."""
    if (name, dtype) not in _made:
        cfg, W = O.random_model(**MODELS[name])
        _made[name, dtype] = cfg, W, VemepelModel(VemepelConfig.from_dict(cfg), {k: torch.tensor(v) for k, v in W.items()}, "cuda", dtype)
    cfg, W, m = _made[name, dtype]
    engine.setdefault("max_tokens", 1024)
    eng = ServingEngine(m, **engine)
    rng = np.random.default_rng(0)
    rng.shuffle(eng.pool.free)
    rng.shuffle(eng.states.free)
    for d in eng.states.data:
        d.normal_()
    return cfg, W, eng


def reference(name, cfg, W, tokens):
    key = (name, tuple(tokens))
    if key not in _refs:
        _refs[key] = O.forward(cfg, W, list(tokens))
    return _refs[key]


def prompt(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


LOGIT_TOL = {F32: 1e-4, BF16: 8e-2}


def close(got, want, dtype, spare=0):
    """f32: every position; bf16: all but a few (a token near the border between two experts may take the other one)."""
    g, w = got.double().cpu().numpy(), np.asarray(want)
    assert g.shape == w.shape and np.isfinite(g).all()
    e = np.sqrt(((g - w) ** 2).mean(-1)) / np.sqrt((w ** 2).mean())
    over = int((e > LOGIT_TOL[dtype]).sum())
    assert over <= (0 if dtype == F32 else max(spare, len(e) // 8)), np.sort(e)[-5:]
    assert np.median(e) < LOGIT_TOL[dtype] / 2


def idle(eng):
    return eng.pool.num_free() == len(eng.pool.pages) and eng.states.num_free() == eng.max_sequences and not eng._fed


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", MODELS)
def test_whole_prompts_and_what_layers_hand_on(name, dtype):
    cfg, W, eng = model_of(name, dtype)
    toks = prompt(cfg, 140, 1)
    taps, trace = [], []
    got = eng.step([StepEntry("a", toks, range(140))], ["a"], taps=taps)
    want = O.forward(cfg, W, toks, trace)
    close(got, want, dtype)
    for t, r in zip(taps, trace):
        close(t, r, dtype)
    assert len(taps) == len(cfg["layers"]) and "a" not in eng and idle(eng)
    close(eng.step([StepEntry("b", toks, [0, 17, 139])], ["b"]), want[[0, 17, 139]], dtype, 1)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", MODELS)
def test_token_by_token_equals_prefill(name, dtype):
    """From the very first token, over several page and chunk borders."""
    cfg, W, eng = model_of(name, dtype)
    assert eng.fast_decode == (dtype == BF16)
    toks = prompt(cfg, 90, 2)
    got = torch.cat([eng.step([StepEntry("a", [t], [0])]) for t in toks])
    close(got, reference(name, cfg, W, toks), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("size", [2, 7, 16, 33, 64])
def test_portions_of_prompts(size, dtype):
    for name in ("layers that differ", "shared keys"):
        cfg, W, eng = model_of(name, dtype)
        toks = prompt(cfg, 135, 3)
        out = []
        for i in range(0, 135, size):
            part = toks[i: i + size]
            out.append(eng.step([StepEntry("a", part, range(len(part)))]))
        close(torch.cat(out), reference(name, cfg, W, toks), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["plain", "shared keys"])
def test_batches_equal_each_request_alone_and_pages_and_slots_are_reused(name, dtype):
    """Unequal requests start together and decode together, shorter ones end earlier; further sets then run on the freed pages and slots."""
    cfg, W, eng = model_of(name, dtype, max_tokens=400, max_sequences=4)
    for wave in range(3):
        lens = {f"{wave}a": (1, 20), f"{wave}b": (40, 3), f"{wave}c": (65, 12), f"{wave}d": (17, 17)}
        toks = {k: prompt(cfg, p + n, wave * 10 + p) for k, (p, n) in lens.items()}
        got = {k: [] for k in lens}

        def take(ids, logits):
            for i, k in enumerate(ids):
                got[k].append(logits[i])
        take(list(lens), eng.step([StepEntry(k, toks[k][:p], [p - 1]) for k, (p, _) in lens.items()]))
        for s in range(20):
            live = [k for k, (p, n) in lens.items() if s < n]
            take(live, eng.step([StepEntry(k, [toks[k][lens[k][0] + s]], [0]) for k in live], [k for k in live if s + 1 == lens[k][1]]))
        assert idle(eng)
        for k, (p, n) in lens.items():
            close(torch.stack(got[k]), reference(name, cfg, W, toks[k])[p - 1: p + n], dtype, 2)


def test_prompts_join_running_sequences_and_large_decode_batches():
    """One step that holds a prompt, a portion and single tokens; then twenty sequences decoding in one step."""
    cfg, W, eng = model_of("plain", BF16, max_tokens=1200)
    toks = {i: prompt(cfg, 30, 50 + i) for i in range(20)}
    eng.step([StepEntry(0, toks[0][:29]), StepEntry(1, toks[1][:10])])
    got = eng.step([StepEntry(0, toks[0][29:], [0]), StepEntry(1, toks[1][10:29], [18]), StepEntry(2, toks[2][:29], [0, 28])])
    want = [reference("plain", cfg, W, toks[0])[29], reference("plain", cfg, W, toks[1])[28], *reference("plain", cfg, W, toks[2])[[0, 28]]]
    close(got, np.stack(want), BF16, 1)
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

    def both(entries):
        x = a.step(entries).clone()                          # the engines share the model's buffers
        return torch.equal(x, b.step(entries))
    for eng in (a, b):
        eng.step([StepEntry("s", toks[:5]), StepEntry("t", toks[:9])])
    for t in toks[5:30]:
        assert both([StepEntry("s", [t], [0]), StepEntry("t", [t], [0])])
    for t in toks[30:]:
        assert both([StepEntry("s", [t], [0])])
    close(b.step([StepEntry("s", [1], [0])]), reference("layers that differ", cfg, W, toks + [1])[-1:], BF16, 1)


def test_long_prompts_and_long_decoding():
    """A long prompt, then hundreds of decoded tokens over many pages and chunks."""
    cfg, W, eng = model_of("plain", BF16, max_tokens=1400)
    toks = prompt(cfg, 1300, 8)
    got = [eng.step([StepEntry("s", toks[:900], [0, 511, 512, 899])])] + [eng.step([StepEntry("s", [t], [0])]) for t in toks[900:]]
    want = reference("plain", cfg, W, toks)
    close(torch.cat(got), want[[0, 511, 512, 899, *range(900, 1300)]], BF16)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_the_previous_token_reaches_across_portions_and_slots(dtype):
    """With shifts of nearly one a token's logits hang on the token before: a lost or foreign state shows in every position that follows a cut."""
    cfg, W = O.random_model(21, kinds="al", mlp="dense")
    for i in range(2):
        W[f"l{i}.shift"][:] = O.bf16(np.full(cfg["width"], 0.95))
    m = VemepelModel(VemepelConfig.from_dict(cfg), {k: torch.tensor(v) for k, v in W.items()}, "cuda", dtype)
    eng = ServingEngine(m, max_tokens=256, max_sequences=2)
    toks, other = prompt(cfg, 40, 1), prompt(cfg, 40, 2)
    want = O.forward(cfg, W, toks)
    foreign = O.forward(cfg, W, [toks[0], other[1], *toks[2:]])
    assert np.abs(foreign[2] - want[2]).max() > 0.3 * np.abs(want[2]).max()
    for wave in range(2):
        eng.step([StepEntry("o", other)])
        got = [eng.step([StepEntry("s", toks[lo:hi], range(hi - lo)), StepEntry("o", other[:2])])[: hi - lo] for lo, hi in ((0, 1), (1, 2), (2, 4), (4, 21))]
        got += [eng.step([StepEntry("s", [t], [0])]) for t in toks[21:]]
        close(torch.cat(got), want, dtype)
        eng.release("s")
        eng.release("o")
    assert idle(eng)


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
    close(x, np.stack([reference("plain", cfg, W, toks[:31])[-1], reference("plain", cfg, W, toks[:30] + other[:1])[-1]]), BF16, 1)
    eng.decode_greedy(["a"], [5], 6)
    assert eng.length("a") == 37
    eng.truncate("a", 31)
    close(eng.step([StepEntry("a", toks[31:], range(19))]), reference("plain", cfg, W, toks)[31:], BF16)
    eng.truncate("b", 0)
    close(eng.step([StepEntry("b", other, range(20))]), reference("plain", cfg, W, other), BF16)
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


def test_checkpoint_directory_and_trace_replay_program(tmp_path):
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
    eng = load_engine(d, "cuda", F32, 64)
    assert eng.generate([toks[:9]], GenerationConfig(max_new_tokens=4)) == [O.greedy(cfg, W, toks[:9], 4)]


def test_random_weights_and_refused_models():
    att = dict(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.25, diff=0.3, mask=dict(size=8))
    lat = dict(heads=2, dim=16, vdim=16, kv_rank=16, scale=0.25)
    cfg = VemepelConfig.pattern("arls", 64, 32, att, lat, dict(lat, rot_dim=8, rot=dict(base=1e4, dims=8)), MoeConfig(4, 2, ExpertConfig(16)), dense_ff=24)
    W = RandomVemepelWeights(cfg)
    assert set(W.keys()) == set(cfg.tensor_shapes()) and cfg.layers[3].mixer.kv_from == 0 and "l0.mlp.act" in W and "l1.mlp.router.b" in W and "l3.mix.k" not in W
    eng = ServingEngine(VemepelModel(cfg, W), max_tokens=32, max_sequences=2)
    assert len(eng.generate([[1, 2, 3]], GenerationConfig(max_new_tokens=4))[0]) == 4 and idle(eng)
    for bad in ({k: W[k] for k in W.keys() if k != "l0.dwa"}, {**{k: W[k] for k in W.keys()}, "l3.mix.k": torch.zeros(64, 32)}):
        with pytest.raises(InvalidArgument):
            VemepelModel(cfg, bad)
    with pytest.raises(InvalidArgument):
        VemepelModel(cfg, W, dtype=torch.float16)
    assert _lib.read_status() == 0
