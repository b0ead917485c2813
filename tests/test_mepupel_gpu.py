"""Mepupel on the device against the plain f64 evaluation in ``mepupel_oracle``: every mechanism by itself, then prompts, portions of prompts, decoding, batches, reuse of pages and
state slots, and generation."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import mepupel_oracle as O
from ferrotorch_b200 import _lib
from ferrotorch_b200.errors import InvalidArgument
from ferrotorch_b200.models import (DecodeState, ExpertConfig, GenerationConfig, MepupelConfig, MepupelModel, MoeConfig, RandomMepupelWeights, RowBatch, ServingEngine, SpecDecodeConfig,
                                    StepEntry, beam_search, generate, speculative_generate)
from ferrotorch_b200.models.llama_infer import _SplitKGemm
from ferrotorch_b200.nn import PagedRowCache, PagePool, StateSlots
from ferrotorch_b200.ops import (DenseGatedWeights, ExpertStack, GqaDecodeBuffers, GqaDims, GqaWeights, LatentDecodeBuffers, LatentDims, LatentWeights, MoeRouting, MoeSmallBuffers, MoeWeights,
                                 RouteRule, SsmDecodeBuffers, SsmDims, SsmWeights, SublayerOutput, dense_gated_rows, gated_act_planes, gqa_attention_decode, gqa_attention_rows,
                                 latent_attention_decode, latent_attention_rows, latent_context, moe_rows, moe_small, pack_head_columns, parallel_embed, parallel_update, state_space_decode,
                                 state_space_rows)
from ferrotorch_b200.ops.latent_attention import rotary_pair_tables
from ferrotorch_b200.ops.streams import padded_vector, round_up

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
TOL = {F32: 5e-6, BF16: 2e-2}
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


def rel(got, want, spare=0):
    """Largest row error (but for ``spare`` rows) relative to the rms of the reference."""
    g, w = got.double().cpu().numpy(), np.asarray(want, dtype=np.float64)
    assert g.shape == w.shape and np.isfinite(g).all()
    return float(np.sort(np.sqrt(((g - w) ** 2).mean(-1)))[len(g) - 1 - spare] / (np.sqrt((w ** 2).mean()) + 1e-30))


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


# -- residual and dense feed-forward -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width", [(1, 5), (3, 2052), (16, 640), (300, 68), (2, 9001)])
def test_residual_with_two_sublayers_side_by_side(dtype, rows, width):
    rng = np.random.default_rng(rows)
    table, ids, ld, eps, mult = rounded(rng.standard_normal((11, width)), dtype), rng.integers(0, 11, rows), round_up(width, 8), 1e-3, 0.37
    x = torch.full((rows, ld), float("nan"), device="cuda")
    h1, h2 = torch.full((2, rows, ld), float("nan"), device="cuda", dtype=dtype)[:, :, :width]
    w1, w2 = rounded(rng.standard_normal((2, width)), F32)
    p1, p2 = padded_vector(dev(w1), "cuda"), padded_vector(dev(w2), "cuda")
    tol = 1e-5 if dtype == F32 else 1e-2
    parallel_embed(torch.as_tensor(ids).cuda(), padded(table, dtype), p1, p2, eps, x, h1, h2, rows)
    want = table[ids]
    assert rel(x[:, :width], want) < 1e-6 and rel(h1, O.rms(want, eps) * w1) < tol and rel(h2, O.rms(want, eps) * w2) < tol
    expert_rows = rounded(rng.standard_normal((3 * rows + 2, width)), dtype)
    row_of = rng.permutation(3 * rows + 2)[: 3 * rows].reshape(rows, 3)
    bias = rounded(rng.standard_normal(width), F32)
    a, b = rng.standard_normal((2, rows, width))
    pa, pb = split_planes(a, 3, rng, pad=rows + 1), split_planes(b, 6, rng, pad=rows + 2)
    sums = [p[:, :rows, :width].double().sum(0).cpu().numpy() for p in (pa, pb)]
    experts = dict(rows=padded(expert_rows, dtype), row_of=torch.as_tensor(row_of, dtype=torch.int32).cuda().contiguous(), top=3)
    mixed = expert_rows[row_of].sum(1)
    for ya, yb, delta, second, store in ((SublayerOutput(planes=pa), SublayerOutput(planes=pb, bias=padded_vector(dev(bias), "cuda")), sums[0] + sums[1] + bias, True, True),
                                         (SublayerOutput(planes=pa), SublayerOutput(**experts), sums[0] + mixed, False, True),
                                         (SublayerOutput(planes=pa, count=3), SublayerOutput(planes=pb, **experts), sums[0] + sums[1] + mixed, True, False),
                                         (SublayerOutput(planes=pa), None, sums[0], True, True)):
        h2.fill_(7.0)
        before = x.clone()
        parallel_update(x, mult, ya, yb, p1, p2 if second else None, eps, h1, h2, rows, width, store)
        new = want + mult * delta
        assert rel(h1, O.rms(new, eps) * w1) < tol and (rel(h2, O.rms(new, eps) * w2) < tol if second else bool((h2 == 7.0).all()))
        if store:
            assert rel(x[:, :width], new) < 5e-6
            want = x[:, :width].double().cpu().numpy()
        else:
            assert torch.equal(x[:, :width], before[:, :width])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width,ff", [(24, 8), (40, 33), (64, 700)])
def test_dense_feed_forward_with_biases(dtype, width, ff):
    rng = np.random.default_rng(ff)
    W = {k: rounded(rng.standard_normal(s) / s[-1] ** 0.5 * 1.5, dtype) for k, s in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))}
    W.update({k + ".b": rounded(rng.standard_normal(n), F32) for k, n in (("gate", ff), ("up", ff), ("down", width))})
    w = DenseGatedWeights.pack(*(torch.tensor(W[k]) for k in ("gate", "up", "down")), "cuda", dtype, "silu", *(torch.tensor(W[k + ".b"]) for k in ("gate", "up", "down")))
    for rows in (1, 5, 130):
        h = rounded(2.0 * rng.standard_normal((rows, width)), dtype)
        y = dense_gated_rows(padded(h, dtype), w)
        assert rel(y.planes[0] + y.bias[:width], O.dense(h, W)) < (1e-5 if dtype == F32 else 2e-2)
    h = rounded(2.0 * rng.standard_normal((7, width)), F32)
    gate, up = h @ W["gate"].T, h @ W["up"].T
    cols = np.zeros((7, w.fp // 8, 2, 8))
    for i, t in enumerate((gate, up)):
        cols[:, :, i] = np.pad(t, ((0, 0), (0, w.fp - ff))).reshape(7, -1, 8)
    out = torch.zeros(16, w.fp, device="cuda", dtype=BF16)
    gated_act_planes(split_planes(cols.reshape(7, -1), 3, rng), 3, 7, w.fp, "silu", out, w.gu_bias)
    assert rel(out[:7, :ff], O.silu(gate + W["gate.b"]) * (up + W["up.b"])) < 1e-2


# -- attention: rotated halves, window, kept first tokens --------------------------------------------------------------------------------
YARN = dict(factor=4.0, original=64, fast=8.0, slow=1.0)


class AttentionRig(Pages):
    """One attention layer fed with projection rows, and the reference."""

    def __init__(self, D, dtype, seed=0, scaling=None, base=700.0):
        self.D, self.dtype, self.rng, self.base, self.scaling = D, dtype, np.random.default_rng(seed), base, scaling
        nq, nk = (D.heads * D.dim, D.kv_heads * D.dim) if D.whole_norm else (D.dim, D.dim)
        self.qn, self.kn = (rounded(1.0 + 0.2 * self.rng.standard_normal(n), F32) for n in (nq, nk))
        self.w = GqaWeights.pack(D, torch.tensor(self.qn), torch.tensor(self.kn), "cuda")
        s = scaling and dict(type="yarn", factor=scaling["factor"], original_max_position=scaling["original"], beta_fast=scaling["fast"], beta_slow=scaling["slow"],
                             attention_factor=0.1 * np.log(scaling["factor"]) + 1.0)
        self.tables = rotary_pair_tables(2048, D.rot_dims, base, "cuda", s)
        super().__init__(D.row, dtype, self.rng)

    def projections(self, n):
        D = self.D
        return {k: rounded(self.rng.standard_normal((n, h, s)), self.dtype) for k, h, s in (("q", D.heads, D.dim), ("k", D.kv_heads, D.dim), ("v", D.kv_heads, D.vdim))}

    def rows(self, P, lo, hi):
        D = self.D
        return torch.cat([pack_head_columns(torch.tensor(P[k][lo:hi]).flatten(1), n, s, "cuda", self.dtype)
                          for k, n, s in (("q", D.heads, D.dim), ("k", D.kv_heads, D.dim), ("v", D.kv_heads, D.vdim))], 1).contiguous()

    def reference(self, P):
        D, n = self.D, P["q"].shape[0]

        def norm(x, w):
            if not D.norm:
                return x
            return (O.rms(x.reshape(n, -1), D.eps) * w).reshape(x.shape) if D.whole_norm else O.rms(x, D.eps) * w
        q, k = (O.rotate_halves(norm(P[a], w), np.arange(n), D.rot_dims, self.base, self.scaling) for a, w in (("q", self.qn), ("k", self.kn)))
        return O.attend(q, k, P["v"], D.scale, O.visible(n, D.window or None, D.keep))

    def heads_of(self, out):
        return out.view(out.shape[0], self.D.heads, self.D.v16)[..., : self.D.vdim].flatten(1)

    def step(self, parts):
        batch = self.batch(parts)
        x = torch.cat([self.rows(*p) for p in parts.values()])
        out = torch.full((x.shape[0], self.D.out_cols), float("nan"), device="cuda", dtype=self.dtype)
        gqa_attention_rows(x, self.w, batch, self.cache.rows[0], *self.tables, None, out)
        self.advance(parts)
        return self.heads_of(out)

    def decode(self, parts, splits=None):
        """One token per sequence: {sequence: (projections, token)}."""
        B, ids = len(parts), list(parts)
        state = self.state(ids)
        planes = split_planes(torch.cat([self.rows(p, t, t + 1) for p, t in parts.values()]).double().cpu().numpy(), 3, self.rng)
        b = GqaDecodeBuffers(self.D, 16, self.blocks * 16, "cuda", splits)
        out = torch.zeros(16, self.D.out_cols, device="cuda", dtype=BF16)
        for _ in range(2):                                  # the second run finds the counters as the first one left them
            gqa_attention_decode(planes, 3, self.w, b, state, self.cache.rows[0], *self.tables, B, 0, out)
        for s in ids:
            self.cache.lengths[s] += 1
        assert not b.counters.any() and not out[B:].any()
        return self.heads_of(out)[:B]


def dims(heads, kv_heads, dim, vdim, rot, window=0, keep=0, norm=False, whole=False):
    return GqaDims(heads, kv_heads, dim, vdim, rot, 1.3 * dim ** -0.5, 1e-4, window, whole, keep=keep, halves=True, norm=norm)


ATTENTION = {
    "one head, no rotation": (dims(1, 1, 8, 8, 0), None),
    "group of four, few kept": (dims(8, 2, 48, 40, 32, window=30, keep=3), YARN),
    "kept tokens over several blocks": (dims(4, 1, 64, 64, 64, window=50, keep=130), YARN),
    "as many kept as seen": (dims(6, 2, 80, 96, 16, window=16, keep=16), None),
    "odd half, odd sizes": (dims(5, 1, 23, 11, 22, window=7, keep=65), YARN),
    "window of one": (dims(4, 2, 32, 16, 12, window=1, keep=1), None),
    "wide heads": (dims(4, 4, 128, 128, 64, window=130, keep=20), dict(factor=40.0, original=4096, fast=32.0, slow=1.0)),
    "wider keys": (dims(2, 1, 300, 60, 200, window=40, keep=9), None),
    "norm per head": (dims(4, 2, 40, 24, 24, window=20, keep=5, norm=True), YARN),
    "norm of the whole projection": (dims(6, 3, 24, 16, 10, norm=True, whole=True), None),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", ATTENTION)
def test_attention_of_ragged_prompts_and_portions(case, dtype):
    D, scaling = ATTENTION[case]
    rig = AttentionRig(D, dtype, 1, scaling)
    P = {s: rig.projections(n) for s, n in (("a", 150), ("b", 1), ("c", 293))}
    rig.open(P)
    got = in_portions(rig.step, P, {"a": [0, 2, 71, 150], "b": [0, 1, 1, 1], "c": [0, 129, 131, 293]})
    for s in P:
        assert rel(got[s], rig.reference(P[s]).reshape(len(got[s]), -1)) < TOL[dtype] * (2 if dtype == F32 else 1), s


@pytest.mark.parametrize("splits", [None, 1, 7])
@pytest.mark.parametrize("case", ATTENTION)
def test_attention_decode_matches_the_whole_sequence(case, splits):
    D, scaling = ATTENTION[case]
    assert D.decode_supported()
    rig = AttentionRig(D, BF16, 2, scaling)
    lens = {"a": 0, "b": 15, "c": 16, "d": 200, "e": 64}
    P = {s: rig.projections(n + 3) for s, n in lens.items()}
    want = {s: rig.reference(p) for s, p in P.items()}
    rig.open(P)
    rig.step({s: (P[s], 0, n) for s, n in lens.items() if n})
    for t in range(3):
        got = rig.decode({s: (P[s], n + t) for s, n in lens.items()}, splits)
        assert rel(got, np.stack([want[s][n + t].reshape(-1) for s, n in lens.items()])) < 2e-2


@pytest.mark.parametrize("heads,kv_heads,window,keep", [(4, 1, 16, 1), (6, 2, 37, 16), (8, 1, 64, 17), (3, 3, 100, 70), (4, 1, 129, 64), (2, 1, 20, 0)])
@pytest.mark.parametrize("target", ["first", "last kept", "first not kept", 63, 64, 130])
def test_one_key_stands_out_while_it_is_visible(heads, kv_heads, window, keep, target):
    """One key meets every query with a score far above all others: its value is the output while the window holds it, and for good if it is one of the kept first tokens. In
    prompts, portions and decoding, around page, block and window borders."""
    target = {"first": 0, "last kept": max(keep - 1, 0), "first not kept": keep}.get(target, target)
    D = GqaDims(heads, kv_heads, 32, 16, 8, 0.6, 1e-6, window, keep=keep, halves=True, norm=False)
    rig = AttentionRig(D, BF16, target)
    n = 270
    P = rig.projections(n)
    P["q"][:] = 0.0
    P["q"][..., 31] = 8.0                                   # beyond the rotated dimensions
    P["k"][..., 31] = 0.0
    P["k"][target] = 0.0
    P["k"][target, :, 31] = 4.0
    want = rig.reference(P)
    for i in range(n):
        seen = target <= i and (i - target < window or target < keep)
        assert (np.abs(want[i] - np.repeat(P["v"][target], heads // kv_heads, 0)).max() < 1e-3) == seen or i == 0
    want = want.reshape(n, -1)
    rig.open(["whole", "parts", "steps"])
    assert rel(rig.step({"whole": (P, 0, n)}), want) < 1e-2
    got = [rig.step({"parts": (P, lo, hi)}) for lo, hi in ((0, 66), (66, 68), (68, 200), (200, n))]
    assert rel(torch.cat(got), want) < 1e-2
    edge = target + window
    lo, hi = max(0, edge - 3), min(n, edge + 4)
    rig.step({"steps": (P, 0, lo)})
    for t in range(lo, hi):
        assert rel(rig.decode({"steps": (P, t)}), want[t].reshape(1, -1)) < 1e-2, t


# -- latent attention: query latents, shared latents, no positions ----------------------------------------------------------------------
LATENT = {"small": (3, 16, 20, 24, 32), "odd sizes": (5, 23, 11, 13, 33), "one head": (1, 8, 8, 1, 1), "wide": (2, 128, 128, 96, 64), "many heads": (34, 32, 16, 40, 48),
          "64": (4, 64, 64, 72, 128), "beyond the tiled kernel": (2, 300, 24, 16, 16), "large latent": (2, 40, 40, 130, 530)}


class LatentRig(Pages):
    """A layer with a latent of its own, and one that reads its latent."""

    def __init__(self, sizes, dtype, seed=0, width=40):
        H, d, dv, qr, r = sizes
        self.dtype, self.rng, self.eps, self.width = dtype, np.random.default_rng(seed), 1e-4, width
        self.m = dict(heads=H, dim=d, vdim=dv, scale=1.2 * d ** -0.5)

        def mat(o, i, s=1.0):
            return rounded(self.rng.standard_normal((o, i)) * s / i ** 0.5, dtype)
        self.W, self.w = [], []
        for own in (True, False):
            W = {"dq": mat(qr, width), "dq.norm": rounded(1 + 0.2 * self.rng.standard_normal(qr), F32), "uq": mat(H * d, qr, 1.5), "uk": mat(H * d, r, 1.5), "uv": mat(H * dv, r), "o": mat(width, H * dv)}
            if own:
                W.update({"dkv": mat(r, width), "dkv.norm": rounded(1 + 0.2 * self.rng.standard_normal(r), F32)})
            D = LatentDims(H, d, 0, dv, r, self.m["scale"], self.eps, qr, own)
            t = {k: torch.tensor(v) for k, v in W.items()}
            self.W.append(W)
            self.w.append(LatentWeights.pack(D, t["uq"], t.get("dkv"), t.get("dkv.norm"), t["uk"], t["uv"], t["o"], "cuda", dtype, dq=t["dq"], q_norm=t["dq.norm"]))
        super().__init__(self.w[0].dims.row, dtype, self.rng, 1024)

    def inputs(self, n):
        return [rounded(self.rng.standard_normal((n, self.width)), self.dtype) for _ in range(2)]

    def reference(self, P):
        c = O.latent_of(P[0], self.W[0], self.eps)
        return np.concatenate([O.latent_mixer(P[i], self.W[i], self.m, self.eps, c) for i in range(2)], 1)

    def step(self, parts):
        batch = self.batch(parts)
        h = [padded(np.concatenate([p[i][lo:hi] for p, lo, hi in parts.values()]), self.dtype) for i in range(2)]
        ctx = latent_context(self.w[0].dims, batch, "cuda", self.dtype) if self.dtype == BF16 else None
        out = [latent_attention_rows(h[i], self.w[i], batch, self.cache.rows[0], None, None, ctx).planes[0] for i in range(2)]
        self.advance(parts)
        return torch.cat(out, 1)

    def decode(self, parts):
        B, ids, out = len(parts), list(parts), []
        state = self.state(ids)
        for i, w in enumerate(self.w):
            h = np.concatenate([p[i][t: t + 1] for p, t in parts.values()])
            proj = [rounded(self.W[i]["dq"], BF16)] + ([rounded(self.W[i]["dkv"], BF16)] if i == 0 else [])
            cols = np.concatenate([np.pad(h @ m.T, ((0, 0), (0, -m.shape[0] % 8))) for m in proj], 1)
            b = LatentDecodeBuffers(w.dims, 16, self.blocks * 16, "cuda")
            a = latent_attention_decode(split_planes(cols, 3, self.rng), 3, w, b, state, self.cache.rows[0], None, None, B, _SplitKGemm(w.uq, "cuda"))
            out.append(a[:B].double() @ w.out.double().t())
        for s in ids:
            self.cache.lengths[s] += 1
        return torch.cat(out, 1)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", LATENT)
def test_latent_attention_of_prompts_and_portions(case, dtype):
    rig = LatentRig(LATENT[case], dtype, 1)
    P = {s: rig.inputs(n) for s, n in (("a", 150), ("b", 1), ("c", 203))}
    rig.open(P)
    got = in_portions(rig.step, P, {"a": [0, 2, 71, 150], "b": [0, 1, 1, 1], "c": [0, 129, 131, 203]})
    for s in P:
        assert rel(got[s], rig.reference(P[s])) < (2e-5 if dtype == F32 else 3e-2), s


@pytest.mark.parametrize("case", [c for c in LATENT if c != "beyond the tiled kernel"])
def test_latent_decode_matches_the_whole_sequence(case):
    rig = LatentRig(LATENT[case], BF16, 2)
    assert all(w.dims.decode_supported() for w in rig.w)
    lens = {"a": 0, "b": 15, "c": 16, "d": 200, "e": 64}
    P = {s: rig.inputs(n + 3) for s, n in lens.items()}
    want = {s: rig.reference(p) for s, p in P.items()}
    rig.open(P)
    rig.step({s: (P[s], 0, n) for s, n in lens.items() if n})
    for t in range(3):
        got = rig.decode({s: (P[s], n + t) for s, n in lens.items()})
        assert rel(got, np.stack([want[s][n + t] for s, n in lens.items()])) < 4e-2


@pytest.mark.parametrize("target", [0, 15, 16, 63, 64, 130])
def test_one_latent_stands_out_however_far_back(target):
    """The input of one token meets every later query with a score far above all others, in the layer that has the latent and in the one that reads it."""
    rig = LatentRig(LATENT["small"], BF16, target)
    m, n = rig.m, 210
    P = rig.inputs(n)
    q = rounded(rig.rng.standard_normal(m["dim"]), BF16)
    for W in rig.W:                                          # queries are one vector, whatever the input; keys of one latent direction point along it
        W["dq"][:] = 0.0
        W["dq"][0, 0] = 1.0
        W["uq"][:] = 0.0
        W["uq"][:, 0] = np.tile(q, m["heads"])
        W["uk"][:] = 0.0
        W["uk"][:, 3] = np.tile(q, m["heads"])
    rig.W[0]["dkv"][3] = 0.0
    rig.W[0]["dkv"][3, 1] = 1.0
    for i in range(2):
        P[i][:, 0] = 1.0
        P[i][:, 1] = 0.0
    P[0][target, 1] = 30.0
    for i, own in enumerate((True, False)):
        t = {k: torch.tensor(v) for k, v in rig.W[i].items()}
        rig.w[i] = LatentWeights.pack(rig.w[i].dims, t["uq"], t.get("dkv"), t.get("dkv.norm"), t["uk"], t["uv"], t["o"], "cuda", BF16, dq=t["dq"], q_norm=t["dq.norm"])
    want = rig.reference(P)
    c = O.latent_of(P[0], rig.W[0], rig.eps)
    alone = c[target] @ rig.W[0]["uv"].T @ rig.W[0]["o"].T
    assert np.abs(want[-1, : rig.width] - alone).max() < 0.05 * np.abs(alone).max()
    rig.open(["whole", "parts", "steps"])
    assert rel(rig.step({"whole": (P, 0, n)}), want) < 3e-2
    assert rel(torch.cat([rig.step({"parts": (P, lo, hi)}) for lo, hi in ((0, 66), (66, 68), (68, n))]), want) < 3e-2
    rig.step({"steps": (P, 0, target + 1)})
    for t in range(target + 1, target + 5):
        assert rel(rig.decode({"steps": (P, t)}), want[t: t + 1]) < 4e-2


# -- state space -------------------------------------------------------------------------------------------------------------------------
class SsmRig(Pages):
    def __init__(self, D, dtype, seed=0, slots=8, dt_mean=-1.0, dt_scale=1.0, a_scale=1.0):
        self.D, self.dtype, self.rng = D, dtype, np.random.default_rng(seed)
        inner, ch = D.heads * D.vdim, D.heads * D.vdim + 2 * D.groups * D.state
        r = self.rng.standard_normal
        self.W = dict(conv=rounded(r((ch, D.taps)) * 1.2 / D.taps ** 0.5, F32), b=rounded(0.2 * r(ch), F32), dt_bias=rounded(dt_mean + r(D.heads), F32), A_log=rounded(a_scale * r(D.heads), F32),
                      D=rounded(1 + 0.3 * r(D.heads), F32), norm=rounded(1 + 0.2 * r(inner), F32))
        self.w = SsmWeights.pack(D, *(torch.tensor(self.W[k]) for k in ("conv", "b", "dt_bias", "A_log", "D", "norm")), "cuda")
        self.dt_scale = dt_scale
        states = StateSlots(slots, [D.state_size], "cuda")
        states.data[0].fill_(float("nan"))                    # what a sequence finds in its slot must not matter
        super().__init__(8, dtype, self.rng, 4096, states)

    def projections(self, n):
        D, r = self.D, lambda *s: rounded(self.rng.standard_normal(s), self.dtype)
        inner = D.heads * D.vdim
        return dict(z=r(n, inner), x=r(n, inner), B=r(n, D.groups * D.state), C=r(n, D.groups * D.state), dt=rounded(self.dt_scale * self.rng.standard_normal((n, D.heads)), F32))

    def reference(self, P):
        """Normed outputs, last states and last inputs of the convolution."""
        D, n = self.D, P["z"].shape[0]
        inner, xbc = D.heads * D.vdim, np.concatenate([P["x"], P["B"], P["C"]], 1)
        x, B, C = np.split(O.silu(O.causal_convolution(xbc, self.W["conv"], self.W["b"])), [inner, inner + D.groups * D.state], 1)
        y, S = O.state_space(x.reshape(n, D.heads, D.vdim), B.reshape(n, D.groups, D.state), C.reshape(n, D.groups, D.state), O.softplus(P["dt"] + self.W["dt_bias"]), self.W["A_log"],
                             self.W["D"])
        last = np.concatenate([np.zeros((D.taps - 1, xbc.shape[1])), xbc])[n:]
        return O.gated_group_norm(y.reshape(n, inner), P["z"], self.W["norm"], D.parts, D.eps), S, last

    def rows(self, P, lo, hi):
        D = self.D
        x = torch.cat([pack_head_columns(torch.tensor(P[k][lo:hi]), n, s, "cuda", F32) for k, n, s in (("z", D.heads, D.vdim), ("x", D.heads, D.vdim), ("B", D.groups, D.state),
                                                                                                        ("C", D.groups, D.state))], 1)
        dt = torch.full((hi - lo, D.h8), float("nan"), device="cuda")
        dt[:, : D.heads] = dev(P["dt"][lo:hi])
        return x, dt

    def heads_of(self, out):
        return out.view(out.shape[0], self.D.heads, self.D.v16)[..., : self.D.vdim].flatten(1)

    def step(self, parts, walk=None):
        batch = self.batch(parts)
        x, dt = (torch.cat(t) for t in zip(*(self.rows(*p) for p in parts.values())))
        out = state_space_rows(x.to(self.dtype), dt, self.w, batch, self.cache.states.data[0], walk)
        self.advance(parts)
        return self.heads_of(out)

    def decode(self, parts):
        B, ids = len(parts), list(parts)
        state = self.state(ids)
        x = torch.cat([torch.cat(self.rows(p, t, t + 1), 1) for p, t in parts.values()])
        x[x.isnan()] = 7.0
        b = SsmDecodeBuffers(self.D, "cuda")
        out = state_space_decode(split_planes(x.double().cpu().numpy(), 3, self.rng), 3, self.w, b, state, self.cache.states.data[0], B)
        for s in ids:
            self.cache.lengths[s] += 1
        assert not out[B:].any() and not b.counters.any()
        return self.heads_of(out)[:B]

    def error(self, s, want):
        """Largest relative error of the state, and of the last inputs of the convolution."""
        D, flat = self.D, self.cache.states.data[0][self.cache.states.slot[s]].double().cpu().numpy()
        n = D.heads * D.n16 * D.v16
        S = flat[:n].reshape(D.heads, D.n16, D.v16)[:, : D.state, : D.vdim]
        if D.taps == 1:
            return np.abs(S - want[1]).max() / np.abs(want[1]).max(), 0.0
        last = flat[n:].reshape(D.taps - 1, D.channels)
        got = np.concatenate([last[:, : D.out_cols].reshape(D.taps - 1, D.heads, D.v16)[..., : D.vdim].reshape(D.taps - 1, -1),
                              last[:, D.out_cols:].reshape(D.taps - 1, 2 * D.groups, D.n16)[..., : D.state].reshape(D.taps - 1, -1)], 1)
        return np.abs(S - want[1]).max() / np.abs(want[1]).max(), np.abs(got - want[2]).max()


SPACES = [SsmDims(2, 16, 16, 1, 4, 1, 1e-5), SsmDims(4, 24, 40, 2, 4, 2, 1e-4), SsmDims(6, 20, 24, 3, 3, 4, 1e-4), SsmDims(1, 96, 128, 1, 2, 1, 1e-6), SsmDims(3, 64, 130, 1, 4, 3, 1e-6),
          SsmDims(9, 5, 3, 9, 1, 5, 1e-3), SsmDims(2, 70, 256, 2, 7, 1, 1e-6), SsmDims(4, 64, 64, 4, 4, 1, 1e-5)]
SPACE_IDS = [f"{d.heads}x{d.vdim}-{d.state}-g{d.groups}-t{d.taps}-p{d.parts}" for d in SPACES]


@pytest.mark.parametrize("form", ["f32", "walk", "tokens"])
@pytest.mark.parametrize("D", SPACES, ids=SPACE_IDS)
def test_state_space_of_prompts_and_portions(D, form):
    """Ragged portions, down to one token, against the recurrence; what is carried to the next portion is exact to 32-bit rounding of what the kernels are given (their operands
    are bf16: outputs of the convolution are rounded)."""
    rig = SsmRig(D, F32 if form == "f32" else BF16, 5)
    P = {"a": rig.projections(200), "b": rig.projections(3), "c": rig.projections(65)}
    rig.open(P)
    got = in_portions(lambda parts: rig.step(parts, None if form == "f32" else form == "walk"), P, {"a": [0, 2, 130, 200], "b": [0, 1, 3, 3], "c": [0, 63, 64, 65]})
    for s in P:
        want = rig.reference(P[s])
        assert rel(got[s], want[0]) < (2e-5 if form == "f32" else 3e-2), s
        state, last = rig.error(s, want)
        assert state < (5e-6 if form == "f32" else 1e-2) and last < 1e-6, s


def space_of(u, D):
    """Convolution outputs as the kernels lay them out -> (x, B, C) in f64."""
    a = u.double().cpu().numpy()
    x = a[:, : D.out_cols].reshape(-1, D.heads, D.v16)[..., : D.vdim]
    B, C = (a[:, D.out_cols + i * D.groups * D.n16:][:, : D.groups * D.n16].reshape(-1, D.groups, D.n16)[..., : D.state] for i in range(2))
    return x, B, C


@pytest.mark.parametrize("rows", [1, 127, 129, 700])
@pytest.mark.parametrize("D", [d for d in SPACES if d.taps > 1], ids=[i for d, i in zip(SPACES, SPACE_IDS) if d.taps > 1])
def test_walked_states_are_exact_for_their_operands(D, rows):
    """The chunked walk against the recurrence on the same bf16 operands: states to 32-bit accuracy (pairs of bf16 numbers hold 16 bits), from zero and from a carried state, in
    one segment and in several."""
    rig = SsmRig(D, BF16, rows)
    rng = rig.rng
    rig.open("s")
    st = rig.cache.states
    slot = st.slot["s"]
    state = None
    for turn in range(2):
        batch = rig.batch({"s": (None, 0, rows)})
        plan = batch.memory_plan(1 if turn else 300)
        u = dev(rng.standard_normal((rows, D.channels)), BF16)
        real = torch.cat([pack_head_columns(torch.ones(1, n * s), n, s, "cuda", F32) for n, s in ((D.heads, D.vdim), (D.groups, D.state), (D.groups, D.state))], 1)
        u = u * real.to(BF16)
        dt = dev(rng.standard_normal((rows, D.h8)))
        o = torch.full((rows, D.out_cols), float("nan"), device="cuda", dtype=BF16)
        sizes, data = (D.heads, D.groups, D.state, D.vdim), st.data[0]
        scratch = torch.full((max(plan.scratch, 1) * D.heads * (D.n16 * D.v16 + 4),), float("nan"), device="cuda")
        vec = (dt, dt.stride(0), rig.w.dt_bias, rig.w.rate, rig.w.skip)
        if plan.scratch:
            _lib.call("ft_ssm_walk", u, rows, *vec, plan.inner, plan.inner.shape[0], *sizes, data, data.stride(0), scratch, None, 0, _lib.S())
            _lib.call("ft_ssm_merge", plan.chains, 1, *sizes, data, data.stride(0), scratch, _lib.S())
        _lib.call("ft_ssm_walk", u, rows, *vec, plan.segments, plan.segments.shape[0], *sizes, data, data.stride(0), scratch, o, 1, _lib.S())
        x, B, C = space_of(u, D)
        d = O.softplus(dt.double().cpu().numpy()[:, : D.heads] + rig.W["dt_bias"])
        y, S = O.state_space(x, B, C, d, rig.W["A_log"], rig.W["D"])
        if state is not None:                                 # the recurrence is linear: add what is left of the carried state
            F = np.exp(np.cumsum(-np.exp(rig.W["A_log"]) * d, 0))
            per = D.heads // D.groups
            y = y + F[:, :, None] * np.einsum("thn,hnv->thv", np.repeat(C, per, 1), state)
            S = S + F[-1][:, None, None] * state
        got = data[slot, : D.heads * D.n16 * D.v16].view(D.heads, D.n16, D.v16).double().cpu().numpy()
        assert np.abs(got[:, : D.state, : D.vdim] - S).max() < 5e-5 * np.abs(S).max()
        assert not got[:, D.state:].any() and not got[:, :, D.vdim:].any()
        assert rel(o.view(rows, D.heads, D.v16)[..., : D.vdim].flatten(1), y.reshape(rows, -1)) < 2e-2
        state = S
        rig.advance({"s": (None, 0, rows)})
    if rows == 700:
        assert plan.scratch > 1


def test_long_prompts_walk_in_segments_beside_short_ones():
    D = SsmDims(2, 32, 48, 1, 4, 2, 1e-5)
    rig = SsmRig(D, BF16, 6, dt_mean=-3.0)
    P, Q = rig.projections(1300), rig.projections(70)
    rig.open("pq")
    want = rig.reference(P)
    a = rig.step({"p": (P, 0, 700)})
    b = rig.step({"q": (Q, 0, 70), "p": (P, 700, 1300)})
    assert rel(torch.cat([a, b[70:]]), want[0]) < 3e-2 and rig.error("p", want)[0] < 1e-2
    assert rel(b[:70], rig.reference(Q)[0]) < 3e-2


@pytest.mark.parametrize("dt_mean,dt_scale,a_scale", [(6.0, 2.0, 1.0), (-8.0, 1.0, 1.0), (0.0, 6.0, 3.0), (30.0, 1.0, 0.1)])
@pytest.mark.parametrize("form", ["f32", "walk", "decode"])
def test_step_sizes_at_their_limits(dt_mean, dt_scale, a_scale, form):
    """States that fade within a token, states that are kept for good, step sizes without a clamp. (Where a token's own product with D nearly cancels, the norm blows up the rounding of
    the convolution's bf16 outputs: a row or two of the walk may be off.)"""
    D = SsmDims(3, 16, 24, 1, 4, 1, 1e-6)
    rig = SsmRig(D, F32 if form == "f32" else BF16, 7, dt_mean=dt_mean, dt_scale=dt_scale, a_scale=a_scale)
    P = rig.projections(150)
    want = rig.reference(P)
    rig.open("s")
    got = torch.cat([rig.decode({"s": (P, t)}) for t in range(150)]) if form == "decode" else rig.step({"s": (P, 0, 150)})
    assert rel(got, want[0], 2 if form == "walk" else 0) < (5e-4 if form == "f32" else 3e-2) and rig.error("s", want)[0] < (1e-4 if form != "walk" else 1e-2)


@pytest.mark.parametrize("target", [0, 1, 127, 128, 255, 256])
@pytest.mark.parametrize("form", ["f32", "walk"])
def test_one_token_is_remembered_across_chunks_segments_and_portions(target, form):
    """Nearly nothing decays and one token's value stands out: every later read-out shows it, wherever chunks, segments and portions end, in prompts and decoding."""
    D = SsmDims(1, 16, 16, 1, 4, 1, 1e-8)
    rig = SsmRig(D, F32 if form == "f32" else BF16, target, dt_mean=-2.0, dt_scale=0.0)
    rig.W["A_log"][:], rig.W["D"][:], rig.W["b"][:] = -9.0, 0.0, 0.0
    rig.W["conv"][:] = 0.0
    rig.W["conv"][:, -1] = 1.0
    rig.w = SsmWeights.pack(D, *(torch.tensor(rig.W[k]) for k in ("conv", "b", "dt_bias", "A_log", "D", "norm")), "cuda")
    P = rig.projections(700)
    P["B"][:], P["C"][:] = 1.0, 1.0
    P["x"] = rounded(P["x"] * 1e-4, rig.dtype)
    P["x"][target] = rounded(4.0 + rig.rng.random(16), rig.dtype)
    want = rig.reference(P)
    rig.open(["whole", "parts", "steps"])
    tol = 1e-3 if form == "f32" else 2e-2
    assert rel(rig.step({"whole": (P, 0, 700)})[target + 1:], want[0][target + 1:]) < tol
    got = torch.cat([rig.step({"parts": (P, lo, hi)}) for lo, hi in ((0, 2), (2, 129), (129, 131), (131, 300), (300, 700))])
    assert rel(got[target + 1:], want[0][target + 1:]) < tol
    if form == "walk":
        rig.step({"steps": (P, 0, target + 1)})
        for t in range(target + 1, target + 6):
            assert rel(rig.decode({"steps": (P, t)}), want[0][t: t + 1]) < tol


@pytest.mark.parametrize("D", SPACES + [SsmDims(2, 200, 400, 1, 4, 8, 1e-6)], ids=SPACE_IDS + ["large"])
def test_state_space_decode(D):
    """Fresh sequences and ones with a prompt behind them; slots that are freed and used again."""
    rig = SsmRig(D, BF16, 8, slots=5)
    for wave in range(2):
        P = {f"{wave}{i}": rig.projections(n + 9) for i, n in enumerate((0, 1, 2, 80, 64))}
        lens = {s: len(p["z"]) - 9 for s, p in P.items()}
        want = {s: rig.reference(p) for s, p in P.items()}
        rig.open(P)
        rig.step({s: (P[s], 0, n) for s, n in lens.items() if n})
        for t in range(9):
            got = rig.decode({s: (P[s], n + t) for s, n in lens.items()})
            assert rel(got, np.stack([want[s][0][n + t] for s, n in lens.items()])) < 3e-2
        for s in P:
            state, last = rig.error(s, want[s])
            assert state < 1e-2 and last < 1e-5
            rig.cache.free_sequence(s)
    assert rig.cache.states.num_free() == 5


# -- mixture of experts ------------------------------------------------------------------------------------------------------------------
def make_moe(dtype, width, experts, top, ff, shared, groups, keep, scale, seed=0):
    rng = np.random.default_rng(seed)
    W = {"router": rounded(rng.standard_normal((experts, width)) * 2 / width ** 0.5, dtype), "correction": rounded(-0.4 + 0.5 * rng.standard_normal(experts), F32)}
    for n, f in [(f"e{i}", ff) for i in range(experts)] + ([("shared", shared)] if shared else []):
        W.update({f"{n}.{k}": rounded(rng.standard_normal(s) * 1.5 / s[1] ** 0.5, dtype) for k, s in (("gate", (f, width)), ("up", (f, width)), ("down", (width, f)))})
    mlp = dict(router=dict(experts=experts, top=top, scale=scale, groups=dict(count=groups, keep=keep) if groups else None), shared=dict(ff=shared) if shared else None)
    stack = lambda names: ExpertStack.pack(*([torch.tensor(W[f"{n}.{k}"]) for n in names] for k in ("gate", "up", "down")), float("inf"), "cuda", dtype)
    w = MoeWeights(padded(W["router"], dtype), stack([f"e{i}" for i in range(experts)]), stack(["shared"]) if shared else None, width, top, form="silu",
                   rule=RouteRule(padded_vector(torch.tensor(W["correction"]), "cuda"), groups, keep, scale))
    return W, mlp, w


def clear_rows(W, mlp, rng, n, dtype):
    """Token rows whose choice of groups and experts is not a close call."""
    rows, r = [], mlp["router"]
    while len(rows) < n:
        h = rounded(rng.standard_normal((1, W["router"].shape[1])), dtype)[0]
        z = W["router"] @ h
        eps = 0.02
        picks = {tuple(sorted(O.route(z + eps * rng.standard_normal(len(z)), W["correction"], r)[0])) for _ in range(12)}
        if len(picks) == 1:
            rows.append(h)
    return np.stack(rows)


MIXTURES = [(40, 8, 3, 24, 16, 4, 2, 1.7), (56, 12, 4, 33, 0, 3, 2, 0.6), (64, 9, 2, 8, 24, 0, 0, 1.0), (32, 6, 1, 40, 40, 6, 3, 2.5), (48, 64, 6, 16, 8, 8, 4, 1.0), (24, 4, 4, 16, 8, 2, 2, 3.0)]


def mixture_of(y, width):
    out = y.planes[: y.count if y.count is not None else y.planes.shape[0], :, :width].double().sum(0) if y.planes is not None else 0.0
    return out + (y.rows.double()[y.row_of.view(-1, y.top).long()].sum(1)[:, :width] if y.rows is not None else 0.0)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", MIXTURES)
def test_mixture_of_any_number_of_tokens(dtype, case):
    W, mlp, w = make_moe(dtype, *case)
    rng = np.random.default_rng(1)
    for n in (1, 17, 300):
        h = clear_rows(W, mlp, rng, n, dtype)
        assert rel(mixture_of(moe_rows(padded(h, dtype), w), case[0]), O.mixture(h, W, mlp)) < (1e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("case", MIXTURES)
def test_mixture_of_a_decode_step(case):
    W, mlp, w = make_moe(BF16, *case)
    rng = np.random.default_rng(2)
    b = MoeSmallBuffers.allocate([w], "cuda")
    b.planes.fill_(float("nan"))
    for n in (1, 2, 8, 9, 16):
        h = clear_rows(W, mlp, rng, n, BF16)
        buf = torch.zeros(16, round_up(case[0], 8), device="cuda", dtype=BF16)[:, : case[0]]
        buf[:n] = dev(h, BF16)
        y = moe_small(buf, w, b, n)
        assert rel(y.planes[: y.count, :n, : case[0]].double().sum(0), O.mixture(h, W, mlp)) < 2e-2


def route_on_device(z, correction, top, groups, keep, scale):
    """Choice and weights of both routers for given logits: the router's weights are the logits, the tokens unit vectors."""
    T, E = z.shape
    assert T <= 16
    zb = rounded(z, BF16)
    rule = RouteRule(dev(correction), groups, keep, scale)
    router = torch.zeros(E, 16, device="cuda", dtype=BF16)
    router[:, :T] = dev(zb.T, BF16)
    h = torch.zeros(16, 16, device="cuda", dtype=BF16)
    h[range(T), range(T)] = 1.0
    stack = ExpertStack.pack([torch.zeros(8, 16)] * E, [torch.zeros(8, 16)] * E, [torch.zeros(16, 8)] * E, float("inf"), "cuda", BF16)
    w = MoeWeights(router, stack, None, 16, top, form="silu", rule=rule)
    r = MoeRouting.choose(h[:T], w)
    many = (r.expert.view(T, top).cpu().numpy(), r.score.view(T, top).cpu().numpy())
    b = MoeSmallBuffers.allocate([w], "cuda")
    moe_small(h, w, b, T)
    n, chosen = int(b.n_active), np.full((T, top), -1)
    for a in range(n):
        for t in range(T):
            p = int(b.pair_of.view(-1, 16)[a, t])
            if p >= 0:
                chosen[t, p % top] = int(b.ids[a])
    return zb, many, (chosen, b.score[: T * top].view(T, top).cpu().numpy())


@pytest.mark.parametrize("groups,keep,top", [(4, 2, 3), (4, 1, 2), (2, 2, 5), (8, 3, 2), (0, 0, 4)])
def test_routing_goes_by_corrected_scores_within_the_best_groups(groups, keep, top):
    rng = np.random.default_rng(groups * 10 + top)
    z, c = 3.0 * rng.standard_normal((16, 8)), -1.5 + rng.standard_normal(8)      # most choice scores are negative
    zb, many, few = route_on_device(z, c, top, groups, keep, 1.3)
    for t in range(16):
        e, w = O.route(zb[t], np.float32(c).astype(np.float64), dict(top=top, scale=1.3, groups=dict(count=groups, keep=keep) if groups else None))
        for got_e, got_w in (many, few):
            assert got_e[t].tolist() == list(e) and np.abs(got_w[t] - w).max() < 1e-5


def test_routing_by_hand():
    """The correction decides the choice but not the weights; a group counts its two best experts, not its best; experts of other groups stay out although all scores are negative."""
    z = np.zeros((1, 6))
    z[0] = [4.0, -4.0, -4.0, 1.0, 1.0, -4.0]                  # two groups of three: one strong expert against two good ones
    _, many, few = route_on_device(z, np.full(6, -2.0), 2, 2, 1, 1.0)
    s = 1 / (1 + np.exp(-1.0))
    for e, w in (many, few):
        assert sorted(e[0]) == [3, 4] and np.allclose(w, 0.5)
    _, many, few = route_on_device(z, np.array([0.0, 0, 0, 0, 0, 5.0]), 2, 2, 1, 2.0)
    for e, w in (many, few):
        assert e[0].tolist() == [5, 3] and np.allclose(w[0], 2.0 * np.array([1 / (1 + np.exp(4.0)), s]) / (1 / (1 + np.exp(4.0)) + s), atol=1e-5)


# -- the model ---------------------------------------------------------------------------------------------------------------------------
MODELS = {
    "plain": dict(seed=1, kinds="mal", scaling=YARN),
    "shared latents": dict(seed=2, kinds="lamlal", overrides={3: dict(kv_from=0), 5: dict(kv_from=0, lat_heads=5, lat_dim=24, q_rank=9)}),
    "state spaces only": dict(seed=3, kinds="mmm", groups=1, norm_groups=4, conv=3, state=40, mlp="dense", ff=33),
    "odd sizes": dict(seed=4, kinds="lamam", vocab=101, width=52, ff=37, heads=5, kv_heads=1, dim=22, vdim=13, rot=6, window=33, keep_first=17, base=300.0, lat_heads=2, lat_dim=21, lat_vdim=9, q_rank=11,
                      kv_rank=19, ssm_heads=3, ssm_vdim=20, state=7, groups=3, norm_groups=5, conv=2, experts=6, top=2, group_count=3, group_keep=1, shared=0, residual_mult=1.0, scaling=YARN),
    "layers that differ": dict(seed=5, kinds="malmla", overrides={0: dict(mlp="dense"), 1: dict(window=70, keep_first=40, rot=0, mlp=None), 2: dict(experts=5, top=4, group_count=0, router_scale=0.5),
                                                                  3: dict(conv=6, ssm_heads=2, ssm_vdim=40, groups=1, norm_groups=1, shared=0), 4: dict(kv_from=2, mlp="dense", ff=9),
                                                                  5: dict(window=1, keep_first=0, heads=2, dim=40, scale=0.3, rot=40, scaling=dict(factor=2.0, original=20, fast=4.0, slow=0.5))}),
    "no feed-forward": dict(seed=6, kinds="alm", mlp=None, residual_mult=0.7),
    "no recurrence": dict(seed=7, kinds="aal", window=0, top=1, experts=4, group_count=2, group_keep=1),
}
_made, _refs = {}, {}


def model_of(name, dtype, **engine):
    """Configuration, weights and engine (models are built once per name and dtype, engines per call); page and slot order are shuffled."""
    if (name, dtype) not in _made:
        cfg, W = O.random_model(**MODELS[name])
        _made[name, dtype] = cfg, W, MepupelModel(MepupelConfig.from_dict(cfg), {k: torch.tensor(v) for k, v in W.items()}, "cuda", dtype)
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
    close(eng.step([StepEntry("b", toks, [0, 17, 139])], ["b"]), want[[0, 17, 139]], dtype, 1)


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
    for name in ("layers that differ", "shared latents"):
        cfg, W, eng = model_of(name, dtype)
        toks = prompt(cfg, 135, 3)
        out = []
        for i in range(0, 135, size):
            part = toks[i: i + size]
            out.append(eng.step([StepEntry("a", part, range(len(part)))]))
        close(torch.cat(out), reference(name, cfg, W, toks), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["plain", "shared latents"])
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
    """The run ahead of the capture leaves no trace in anybody's state; sublayers on two streams give the same bits as one after another."""
    cfg, W, a = model_of("layers that differ", BF16)
    _, _, b = model_of("layers that differ", BF16, use_graph=False)
    toks = prompt(cfg, 60, 6)

    def both(entries):
        x = a.step(entries)
        b.model.side_by_side = len(entries) == 2
        y = b.step(entries)
        b.model.side_by_side = True
        return torch.equal(x, y)
    for eng in (a, b):
        eng.step([StepEntry("s", toks[:5]), StepEntry("t", toks[:9])])
    for t in toks[5:30]:
        assert both([StepEntry("s", [t], [0]), StepEntry("t", [t], [0])])
    for t in toks[30:]:
        assert both([StepEntry("s", [t], [0])])
    close(a.step([StepEntry("s", [1], [0])]), reference("layers that differ", cfg, W, toks + [1])[-1:], BF16, 1)


def test_long_prompts_and_long_decoding():
    """A prompt that walks in segments, then hundreds of decoded tokens over many pages."""
    cfg, W, eng = model_of("plain", BF16, max_tokens=1400)
    toks = prompt(cfg, 1300, 8)
    got = [eng.step([StepEntry("s", toks[:900], [0, 511, 512, 899])])] + [eng.step([StepEntry("s", [t], [0])]) for t in toks[900:]]
    want = reference("plain", cfg, W, toks)
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
    att = dict(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.25, rot=dict(base=1e4, dims=8), mask=dict(size=8, keep_first=2))
    cfg = MepupelConfig.pattern("mals", 64, 32, dict(heads=2, vdim=16, state=16, groups=1, norm_groups=2, conv=4), att, dict(heads=2, dim=16, vdim=16, q_rank=16, kv_rank=16, scale=0.25),
                                MoeConfig(4, 2, ExpertConfig(16), ExpertConfig(16), 2, 1, 1.5), first_ff=24)
    W = RandomMepupelWeights(cfg)
    assert set(W.keys()) == set(cfg.tensor_shapes()) and cfg.layers[3].mixer.kv_from == 2 and "l0.mlp.gate.b" in W and "l3.mix.dkv" not in W
    eng = ServingEngine(MepupelModel(cfg, W), max_tokens=32, max_sequences=2)
    assert len(eng.generate([[1, 2, 3]], GenerationConfig(max_new_tokens=4))[0]) == 4 and idle(eng)
    for bad in ({k: W[k] for k in W.keys() if k != "l0.mix.A_log"}, {**{k: W[k] for k in W.keys()}, "l3.mix.dkv": torch.zeros(16, 32)}):
        with pytest.raises(InvalidArgument):
            MepupelModel(cfg, bad)
    with pytest.raises(InvalidArgument):
        MepupelModel(cfg, W, dtype=torch.float16)
