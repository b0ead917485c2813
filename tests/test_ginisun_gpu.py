"""Ginisun on the device against the plain f64 evaluation in ``ginisun_oracle``: every mechanism by itself, then prompts, portions of prompts, decoding,
batches, page reuse and generation."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import ginisun_oracle as O
from ferrotorch_b200 import _lib
from ferrotorch_b200.models import GenerationConfig, GinisunConfig, GinisunModel, RandomGinisunWeights, ServingEngine, StepEntry, beam_search, generate
from ferrotorch_b200.models import SpecDecodeConfig, generate_with_streamer, speculative_generate
from ferrotorch_b200.ops import latent_attention as LA
from ferrotorch_b200.ops import moe as M
from ferrotorch_b200.ops import streams as ST
from ferrotorch_b200.ops import (DynamicTanhWeights, HyperWeights, LatentDecodeBuffers, LatentDims, LatentWeights, MoeRouting, MoeSmallBuffers, MoeWeights, ExpertStack,
                                 SublayerOutput, absorb_queries, dynamic_tanh, expand_values, grouped_linear, hyper_embed, hyper_update, moe_rows, moe_small)

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
TOL = {F32: 3e-6, BF16: 2e-2}


def dev(a, dtype=F32):
    return torch.as_tensor(np.asarray(a, dtype=np.float32)).cuda().to(dtype)


def padded(a, dtype, multiple=8):
    t = dev(a, dtype)
    buf = torch.full((t.shape[0], ST.round_up(t.shape[1], multiple)), float("nan"), device="cuda", dtype=dtype)
    buf[:, : t.shape[1]] = t
    return buf[:, : t.shape[1]]


def rel(got, want):
    """Largest row error relative to the rms of the reference."""
    g, w = got.double().cpu().numpy(), np.asarray(want, dtype=np.float64)
    assert g.shape == w.shape and np.isfinite(g).all()
    return float(np.sqrt(((g - w) ** 2).mean(-1)).max() / (np.sqrt((w ** 2).mean()) + 1e-30))


def rounded(a, dtype):
    """f64 values of the device copy (so that input rounding is not part of the error)."""
    return dev(a, dtype).double().cpu().numpy()


# -- streams and norm ------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width", [(1, 5), (7, 64), (33, 2052)])
def test_dynamic_tanh(dtype, rows, width):
    rng = np.random.default_rng(width)
    x, w, b = rounded(rng.standard_normal((rows, width)) * 3, dtype), rng.standard_normal(width), rng.standard_normal(width)
    wt = DynamicTanhWeights.from_tensors(torch.tensor(0.7), torch.tensor(w), torch.tensor(b), "cuda")
    assert rel(dynamic_tanh(padded(x, dtype), wt), O.dynamic_tanh(x, 0.7, w, b)) < TOL[dtype]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n,rows,width", [(1, 3, 40), (2, 9, 12), (3, 1, 300), (4, 70, 512), (6, 5, 21)])
def test_streams_start_update_and_end(dtype, n, rows, width):
    rng = np.random.default_rng(n * 100 + rows)
    table, ids = rounded(rng.standard_normal((11, width)), dtype), rng.integers(0, 11, rows)
    vec = {k: (0.4 + rng.random(), rng.standard_normal(width), rng.standard_normal(width)) for k in "abc"}
    N = {k: DynamicTanhWeights.from_tensors(torch.tensor(a), torch.tensor(w), torch.tensor(b), "cuda") for k, (a, w, b) in vec.items()}
    inp, mix, out, inp2 = rng.standard_normal(n), rng.standard_normal((n, n)), rng.standard_normal(n), rng.standard_normal(n)
    hw = HyperWeights.from_tensors(torch.tensor(inp), torch.tensor(mix), torch.tensor(out), "cuda")
    ld = ST.round_up(width, 8)
    x = torch.full((rows, n, ld), float("nan"), device="cuda")
    h = torch.full((rows, ld), float("nan"), device="cuda", dtype=dtype)[:, :width]
    hyper_embed(torch.tensor(ids).cuda(), padded(table, dtype), N["a"], x, hw.inp, N["b"], h, rows, width)
    x0 = O.dynamic_tanh(table[ids], *vec["a"])
    s = np.stack([x0] * n)
    assert rel(x[:, :, :width].transpose(0, 1).reshape(-1, width), s.reshape(-1, width)) < 3e-6
    assert rel(h, O.dynamic_tanh(O.connect_in(s, inp), *vec["b"])) < TOL[dtype]
    # the update takes planes, picked rows, or both; streams differ from one another after the first one
    for planes, top in ((2, 0), (0, 3), (1, 2)):
        p = rng.standard_normal((planes, rows, width))
        pool, pick = rounded(rng.standard_normal((rows * 4, width)), dtype), rng.integers(0, rows * 4, (rows, max(top, 1)))
        y = p.sum(0) + (pool[pick].sum(1) if top else 0.0)
        pd = torch.zeros(max(planes, 1), rows, ld, device="cuda")
        pd[:planes, :, :width] = dev(p)
        sub = SublayerOutput(planes=pd if planes else None, count=planes, rows=padded(pool, dtype) if top else None,
                             row_of=torch.tensor(pick[:, :top], dtype=torch.int32).cuda().contiguous(), top=top)
        hyper_update(x, hw, sub, dev(inp2), N["c"], h, rows, width)
        s = O.connect_out(s, y, mix, out)
        assert rel(x[:, :, :width].transpose(0, 1).reshape(-1, width), s.reshape(-1, width)) < 1e-5
        assert rel(h, O.dynamic_tanh(O.connect_in(s, inp2), *vec["c"])) < TOL[dtype]
    before = x.clone()
    hyper_update(x, hw, SublayerOutput(planes=pd, count=1), None, N["a"], h, rows, width, store=False)
    last = O.connect_out(s, p[0], mix, out).sum(0)
    assert rel(h, O.dynamic_tanh(last, *vec["a"])) < TOL[dtype]
    assert torch.equal(x[:, :, :width], before[:, :, :width])


# -- latent attention ------------------------------------------------------------------------------------------------------------------
DIMS = [dict(heads=3, dim=16, rot_dim=8, vdim=24, rank=40), dict(heads=5, dim=20, rot_dim=6, vdim=12, rank=33), dict(heads=2, dim=64, rot_dim=64, vdim=64, rank=128),
        dict(heads=4, dim=128, rot_dim=64, vdim=128, rank=512), dict(heads=2, dim=96, rot_dim=32, vdim=72, rank=64), dict(heads=1, dim=160, rot_dim=64, vdim=200, rank=96),
        dict(heads=40, dim=24, rot_dim=16, vdim=16, rank=48), dict(heads=17, dim=8, rot_dim=2, vdim=8, rank=8), dict(heads=2, dim=320, rot_dim=64, vdim=128, rank=64)]


def make_attention(D, width=48, seed=0, scale=None):
    rng = np.random.default_rng(seed)
    H, dn, dr, dv, r = D["heads"], D["dim"], D["rot_dim"], D["vdim"], D["rank"]
    W = {"q": rng.standard_normal((H * (dn + dr), width)) / 5, "dkv": rng.standard_normal((r + dr, width)) / 5, "dkv.norm": 1 + 0.2 * rng.standard_normal(r),
         "uk": rng.standard_normal((H * dn, r)) / r ** 0.5, "uv": rng.standard_normal((H * dv, r)) / r ** 0.5, "o": rng.standard_normal((width, H * dv)) / (H * dv) ** 0.5}
    W = {k: rounded(v, BF16) for k, v in W.items()}
    mixer = dict(heads=H, dim=dn, rot_dim=dr, vdim=dv, kv_rank=r, scale=scale or (dn + dr) ** -0.5, rot=dict(base=1000.0, dims=dr))
    return W, mixer, LatentDims(H, dn, dr, dv, r, mixer["scale"], 1e-5)


class Bench:
    """One latent-attention layer with a page cache whose free list is shuffled, so that sequences get scattered pages."""

    def __init__(self, D, dtype, pages=64, **kw):
        from ferrotorch_b200.nn import PagedRowCache, PagePool
        self.W, self.mixer, self.dims = make_attention(D, **kw)
        self.dtype = dtype
        self.w = LatentWeights.pack(self.dims, *(torch.tensor(self.W[k]) for k in ("q", "dkv", "dkv.norm", "uk", "uv", "o")), "cuda", dtype)
        self.pool = PagePool(pages, 16)
        np.random.default_rng(1).shuffle(self.pool.free)
        self.cache = PagedRowCache(self.pool, [self.dims.row], "cuda", dtype)
        self.pages = pages
        self.cos, self.sin = LA.rotary_pair_tables(pages * 16, self.dims.rot_dim, 1000.0, "cuda")

    def reference(self, h):
        return O.latent_attention(h, self.W, self.mixer, 1e-5)

    def run(self, parts):
        """``parts``: {sequence: new rows}; returns the outputs by sequence."""
        from ferrotorch_b200.models import RowBatch
        entries = [StepEntry(k, [0] * len(h)) for k, h in parts.items()]
        for e in entries:
            if e.id not in self.cache.tables:
                self.cache.add_sequence(e.id)
            self.cache.reserve(e.id, self.cache.lengths[e.id] + len(e.tokens))
        b = RowBatch(entries, self.cache, "cuda", self.pages)
        h = padded(np.concatenate(list(parts.values())), self.dtype)
        y = LA.latent_attention_rows(h, self.w, b, self.cache.rows[0], self.cos, self.sin).planes[0]
        out, at = {}, 0
        for e in entries:
            self.cache.lengths[e.id] += len(e.tokens)
            out[e.id] = y[at: at + len(e.tokens)]
            at += len(e.tokens)
        return out


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("D", DIMS, ids=lambda d: "-".join(map(str, d.values())))
def test_latent_attention_of_ragged_prompts_and_portions(dtype, D):
    B = Bench(D, dtype)
    rng = np.random.default_rng(3)
    seqs = {n: rounded(rng.standard_normal((n, 48)), dtype) for n in (1, 16, 23, 150, 290)}
    ref = {n: B.reference(h) for n, h in seqs.items()}
    got = B.run(seqs)
    for n in seqs:
        assert rel(got[n], ref[n]) < (1e-5 if dtype == F32 else 2.5e-2), n
    # the same in portions, next to another sequence's portions, after the first ones were freed
    for n in seqs:
        B.cache.free_sequence(n)
    cuts = {150: [0, 2, 16, 33, 64, 129, 150], 290: [0, 128, 130, 131, 257, 289, 290]}
    for i in range(6):
        got = B.run({n: seqs[n][c[i]: c[i + 1]] for n, c in cuts.items()})
        for n, c in cuts.items():
            assert rel(got[n], ref[n][c[i]: c[i + 1]]) < (1e-5 if dtype == F32 else 2.5e-2), (n, c[i])


@pytest.mark.parametrize("tokens", [1, 9, 16])
@pytest.mark.parametrize("D", [d for d in DIMS if d["dim"] < 160], ids=lambda d: "-".join(map(str, d.values())))
def test_latent_decode_matches_the_whole_sequence(D, tokens):
    B = Bench(D, BF16, pages=320)
    assert B.dims.decode_supported()
    rng = np.random.default_rng(5)
    lens = [1, 2, 15, 16, 17, 31, 63, 64, 65, 127, 128, 129, 191, 193, 257, 300][-tokens:]
    seqs = [rounded(rng.standard_normal((n, 48)), BF16) for n in lens]
    for i, h in enumerate(seqs):
        if lens[i] > 1:
            B.run({i: h[:-1]})
        else:
            B.cache.add_sequence(i)
        B.cache.reserve(i, lens[i])
    from ferrotorch_b200.models import DecodeState
    from ferrotorch_b200.models.llama_infer import _SplitKGemm
    st = DecodeState("cuda", 20)
    st.load([0] * tokens, [n - 1 for n in lens], B.cache.block_table(range(tokens), 20))
    g, go = _SplitKGemm(B.w.proj, "cuda"), _SplitKGemm(B.w.out, "cuda")
    h = torch.zeros(16, 48, device="cuda", dtype=BF16)
    h[:tokens] = dev(np.stack([s[-1] for s in seqs]), BF16)
    want = np.stack([B.reference(s)[-1] for s in seqs])
    for splits in (None, 1, 3, 64):
        buf = LatentDecodeBuffers(B.dims, 16, 320, "cuda", splits)
        g(h)
        go(LA.latent_attention_decode(g.planes, g.splits, B.w, buf, st, B.cache.rows[0], B.cos, B.sin, tokens))
        assert rel(go.planes.sum(0)[:tokens, :48], want) < 3e-2, splits


def _standing_out(n, target, D, rng):
    """Queries and cached rows of one head group where every query at or after ``target`` looks at that key and at nothing else."""
    row, r16 = D.row, D.r16
    rows = rng.standard_normal((n, row)) * 0.05
    rows[:, D.rank: r16] = 0
    rows[:, r16 + D.rot_dim:] = 0
    key = np.zeros(row)
    key[: D.rank] = rng.choice([-1.0, 1.0], D.rank)
    key[r16: r16 + D.rot_dim] = rng.choice([-1.0, 1.0], D.rot_dim)
    rows[target] = key
    return rows, key * (60.0 / (D.rank + D.rot_dim) / D.scale)


@pytest.mark.parametrize("heads,rank", [(3, 32), (20, 64)])
def test_one_far_key_is_found_wherever_it_lies(heads, rank):
    """A single cached row carries all the weight: at page borders, chunk borders, split borders, the first and the last token."""
    D = LatentDims(heads, 16, 16, 16, rank, 0.2, 1e-5)
    rng = np.random.default_rng(9)
    n = 517
    perm = torch.tensor(rng.permutation(40)[:33].astype(np.int32)).cuda().view(1, 33)
    for target in (0, 1, 15, 16, 17, 31, 63, 64, 65, 127, 128, 255, 256, 511, 512, 515, 516):
        rows, q = _standing_out(n, target, D, rng)
        rows = rounded(rows, BF16)
        for dtype in (F32, BF16):
            store = torch.full((40, 16, D.row), float("nan"), device="cuda", dtype=dtype)
            flat = torch.zeros(33 * 16, D.row, device="cuda", dtype=dtype)
            flat[:n] = dev(rows, dtype)
            store[perm[0].long()] = flat.view(33, 16, D.row)
            qd = dev(np.broadcast_to(q, (1, heads, D.row)), dtype).contiguous()
            out = torch.zeros(1, heads, D.r16, device="cuda", dtype=dtype)
            pos = torch.tensor([n - 1], dtype=torch.int32).cuda()
            _lib.call("ft_latent_rows", qd, store, perm, 33, None, pos, 1, heads, D.rot_dim, D.rank, D.scale, out, int(dtype == F32), _lib.S())
            assert rel(out[0, :, : D.rank], np.broadcast_to(rows[target, : D.rank], (heads, D.rank))) < 1e-2, (target, dtype)
            if target:                                                   # the query one token earlier than the key must not see it
                _lib.call("ft_latent_rows", qd, store, perm, 33, None, torch.tensor([target - 1], dtype=torch.int32).cuda(), 1, heads, D.rot_dim, D.rank, D.scale, out,
                          int(dtype == F32), _lib.S())
                assert float(out.float().abs().max()) < 0.5
        for splits in (1, 5, 9, 33):
            b = LatentDecodeBuffers(D, 1, 528, "cuda", splits)
            lens = torch.tensor([n], dtype=torch.int32).cuda()
            _lib.call("ft_latent_decode", qd, store, perm, 33, lens, 1, heads, D.rot_dim, D.rank, D.scale, splits, b.mt, b.ws, _lib.S())
            _lib.call("ft_latent_combine", b.ws, 1, heads, D.rank, splits, b.mt, out, _lib.S())
            assert rel(out[0, :, : D.rank], np.broadcast_to(rows[target, : D.rank], (heads, D.rank))) < 1e-2, (target, splits)


@pytest.mark.parametrize("dn,dr,dv", [(16, 16, 16), (64, 32, 64), (128, 64, 128), (64, 64, 128), (128, 64, 40), (192, 64, 192)])
def test_one_far_key_in_prompts(dn, dr, dv):
    """The tiled prompt kernel on two sequences: every query from the target on returns the target's value, every earlier one does not see it."""
    rng = np.random.default_rng(dn + dv)
    H, lens = 2, [300, 421]
    D = LatentDims(H, dn, dr, dv, 32, 0.2, 1e-5)
    tile = D.flash_tile()
    assert tile == _lib.kernels().ft_latent_flash_tile(dn, dr, dv) and tile in (128, 256)
    T = sum(lens)
    tiles = [(o + m, min(tile, n - m), m, o) for o, n in ((0, lens[0]), (lens[0], lens[1])) for m in range(0, n, tile)]
    tl = torch.tensor(tiles, dtype=torch.int32).cuda()
    for target in (0, 1, 63, 64, 65, 127, 128, 129, 255, 256, 257, 299):
        direction = rng.choice([-1.0, 1.0], (H, dn))
        rot = rng.choice([-1.0, 1.0], dr)
        c = 60.0 / (dn + dr) / D.scale
        q = np.zeros((T, H, D.dim8 + D.rot8))
        q[:, :, :dn], q[:, :, D.dim8: D.dim8 + dr] = direction * c, rot * c
        k, v, kr = rng.standard_normal((T, H, D.dim8)) * 0.05, rng.standard_normal((T, H, D.v8)), rng.standard_normal((T, D.rot8)) * 0.05
        for o in (0, lens[0]):
            k[o + target, :, :dn], kr[o + target, :dr] = direction, rot
        v = rounded(v, BF16)
        qd, kvd, krd = dev(q.reshape(T, -1), BF16), dev(np.concatenate([k.reshape(T, -1), v.reshape(T, -1)], 1), BF16), dev(kr, BF16)
        out = torch.full((T, H * D.v8), float("nan"), device="cuda", dtype=BF16)
        _lib.call("ft_latent_flash", qd, qd.stride(0), T, kvd, kvd.stride(0), krd, krd.stride(0), T, tl, len(tiles), H, dn, dr, dv, D.scale, None, 0, 0, out, out.stride(0), _lib.S())
        got = out.view(T, H, D.v8)[:, :, :dv].float().cpu().numpy()
        assert np.isfinite(got).all()
        for o, n in ((0, lens[0]), (lens[0], lens[1])):
            assert np.abs(got[o + target: o + n] - v[o + target, :, :dv]).max() < 2e-2, target
            if target > 8:
                assert np.abs(got[o + target - 1] - v[o + target, :, :dv]).max() > 0.1, target


def test_absorbed_form_equals_expanded_form():
    for dtype in (F32, BF16):
        B = Bench(DIMS[1], dtype)
        D, T = B.dims, 9
        rng = np.random.default_rng(2)
        q = padded(rng.standard_normal((T, D.proj_cols)), dtype)
        q.nan_to_num_()
        full = absorb_queries(q, B.w)
        heads = q[:, : D.q_cols].double().cpu().numpy().reshape(T, D.heads, -1)
        want = np.einsum("thd,hdr->thr", heads[:, :, : D.dim], B.W["uk"].reshape(D.heads, D.dim, D.rank))
        assert rel(full[:, :, : D.rank].reshape(-1, D.rank), want.reshape(-1, D.rank)) < (1e-5 if dtype == F32 else 1e-2)
        assert torch.equal(full[:, :, D.r16: D.r16 + D.rot_dim], q[:, : D.q_cols].unflatten(1, (D.heads, -1))[:, :, D.dim8: D.dim8 + D.rot_dim])
        lat = torch.zeros(T, D.heads, D.r16, device="cuda", dtype=dtype)
        lat[:, :, : D.rank] = dev(rng.standard_normal((T, D.heads, D.rank)), dtype)
        want = np.einsum("thr,hvr->thv", lat[:, :, : D.rank].double().cpu().numpy(), B.W["uv"].reshape(D.heads, D.vdim, D.rank))
        got = expand_values(lat, B.w).view(T, D.heads, D.v8)[:, :, : D.vdim]
        assert rel(got.reshape(-1, D.vdim), want.reshape(-1, D.vdim)) < (1e-5 if dtype == F32 else 1e-2)


# -- mixture of experts ----------------------------------------------------------------------------------------------------------------
def make_moe(width, experts, top, ff, shared, dtype, limit=1.25, shared_limit=0.6, seed=0):
    rng = np.random.default_rng(seed)
    W = {"router": rng.standard_normal((experts, width)) * 2 / width ** 0.5}
    for nm, f in [(f"e{i}", ff) for i in range(experts)] + ([("shared", shared)] if shared else []):
        W[nm + ".gate"], W[nm + ".up"] = (rng.standard_normal((f, width)) * 2 / width ** 0.5 for _ in range(2))
        W[nm + ".down"] = rng.standard_normal((width, f)) / f ** 0.5
    W = {k: rounded(v, BF16) for k, v in W.items()}
    cfg = dict(router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit))
    if shared:
        cfg["shared"] = dict(ff=shared, limit=shared_limit)
    t = {k: torch.tensor(v) for k, v in W.items()}

    def stack(names, lim):
        return ExpertStack.pack(*[[t[f"{n}.{k}"] for n in names] for k in ("gate", "up", "down")], lim, "cuda", dtype)
    router = torch.zeros(experts, ST.round_up(width, 8), device="cuda", dtype=dtype)
    router[:, :width] = t["router"].cuda().to(dtype)
    mw = MoeWeights(router[:, :width], stack([f"e{i}" for i in range(experts)], limit), stack(["shared"], shared_limit) if shared else None, width, top)
    return W, cfg, mw


def moe_result(sub, tokens, width):
    y = torch.zeros(tokens, width, device="cuda", dtype=torch.float64)
    if sub.planes is not None:
        n = sub.count if sub.count is not None else sub.planes.shape[0]
        y += sub.planes[:n, :tokens, :width].double().sum(0)
    if sub.rows is not None:
        y += sub.rows[sub.row_of.view(tokens, sub.top).long()][..., :width].double().sum(1)
    return y


def clear_tokens(rng, W, tokens, width, top, dtype):
    """Token rows without close calls between the chosen experts and the next one."""
    out = []
    while len(out) < tokens:
        h = rounded(rng.standard_normal((1, width)), dtype)
        z = np.sort(h @ W["router"].T)[0][::-1]
        if top == len(z) or z[top - 1] - z[top] > 1e-3:
            out.append(h[0])
    return np.stack(out)


MOES = [(48, 4, 1, 24, 40), (64, 7, 3, 20, 0), (100, 5, 5, 33, 17), (256, 130, 8, 64, 96), (40, 1, 1, 16, 16), (1024, 9, 2, 512, 768)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width,experts,top,ff,shared", MOES)
def test_mixture_of_any_number_of_tokens(dtype, width, experts, top, ff, shared):
    W, cfg, mw = make_moe(width, experts, top, ff, shared, dtype)
    rng = np.random.default_rng(7)
    for tokens in (1, 5, 200):
        h = clear_tokens(rng, W, tokens, width, top, dtype)
        hd = padded(h, dtype)
        r = MoeRouting.choose(hd, mw)
        want_e, want_s = O.route(h, W["router"], top)
        assert np.array_equal(r.expert.view(tokens, top).cpu().numpy(), want_e)
        assert np.abs(r.score.view(tokens, top).cpu().numpy() - want_s).max() < (1e-6 if dtype == F32 else 1e-4)
        rows = r.start.long()[r.expert.long()] + r.pos
        assert rows.unique().numel() == tokens * top and int(rows.max()) < r.tile_group.numel() * 128
        assert torch.equal(r.tile_group[rows // 128], r.expert)
        assert rel(moe_result(moe_rows(hd, mw), tokens, width), O.mixture(h, W, cfg)) < (1e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("width,experts,top,ff,shared", MOES)
def test_mixture_of_a_decode_step(width, experts, top, ff, shared):
    W, cfg, mw = make_moe(width, experts, top, ff, shared, BF16)
    assert mw.small_supported()
    rng = np.random.default_rng(8)
    buf = MoeSmallBuffers.allocate([mw], "cuda")
    h16 = torch.full((16, ST.round_up(width, 8)), float("nan"), device="cuda", dtype=BF16)[:, :width]
    for tokens in (1, 2, 8, 9, 16, 3):
        h = clear_tokens(rng, W, tokens, width, top, BF16)
        h16[:tokens] = dev(h, BF16)
        got = moe_result(moe_small(h16, mw, buf, tokens), tokens, width)
        assert rel(got, O.mixture(h, W, cfg)) < 2e-2, tokens
        chosen = np.unique(O.route(h, W["router"], top)[0])
        n = int(buf.n_active)
        assert buf.ids[:n].tolist() == chosen.tolist() and int(buf.cnt[:n].sum()) == tokens * top and int(buf.counter) == 0
    # all tokens on the same experts: every column of the tensor tile in use
    h16[:] = dev(h[:1], BF16)
    assert rel(moe_result(moe_small(h16, mw, buf, 16), 16, width), np.repeat(O.mixture(h[:1], W, cfg), 16, 0)) < 2e-2
    assert int(buf.n_active) == top


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_limits_clip_gate_from_above_and_up_on_both_sides(dtype):
    """Large projections of either sign: the gate is bounded above only."""
    W, cfg, mw = make_moe(32, 2, 1, 16, 16, dtype, limit=0.8, shared_limit=2.5)
    rng = np.random.default_rng(1)
    h = clear_tokens(rng, W, 40, 32, 1, dtype)
    h = rounded(h * 6, dtype)
    assert rel(moe_result(moe_rows(padded(h, dtype), mw), 40, 32), O.mixture(h, W, cfg)) < (1e-5 if dtype == F32 else 2e-2)


def test_equal_scores_choose_the_lower_expert():
    W, cfg, mw = make_moe(16, 6, 2, 8, 0, F32)
    mw.router.zero_()
    r = MoeRouting.choose(padded(np.ones((3, 16)), F32), mw)
    assert r.expert.tolist() == [0, 1] * 3 and torch.allclose(r.score, torch.full((6,), 0.5, device="cuda"))


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_grouped_product_skips_unused_tiles(dtype):
    rng = np.random.default_rng(4)
    x, w = rng.standard_normal((4 * 128, 40)), rng.standard_normal((3, 32, 64))
    xd, wd = dev(x, dtype), dev(w, dtype)
    out = torch.full((512, 24), 7.0, device="cuda", dtype=dtype)
    grouped_linear(xd, wd, torch.tensor([2, -1, 0, 2], dtype=torch.int32).cuda(), 24, 40, out)
    for i, g in enumerate([2, None, 0, 2]):
        part = out[i * 128: (i + 1) * 128]
        if g is None:
            assert bool((part == 7.0).all())
        else:
            ref = xd[i * 128: (i + 1) * 128].double() @ wd[g, :24, :40].double().t()
            assert rel(part, ref.cpu().numpy()) < (1e-5 if dtype == F32 else 1e-2)


# -- the model -------------------------------------------------------------------------------------------------------------------------
MODELS = {
    "plain": dict(seed=1),
    "one stream, top one": dict(seed=2, streams=1, top=1, heads=(4,)),
    "odd sizes": dict(seed=3, vocab=101, width=52, heads=(3, 5, 1), dim=20, rot_dim=6, vdim=12, kv_rank=33, experts=3, top=3, ff=19, shared_ff=11, streams=5),
    "layers that differ": dict(seed=4, heads=(2, 4, 3), overrides={0: dict(mlp=False), 1: dict(dim=24, rot_dim=12, vdim=40, kv_rank=16, base=500.0, experts=9, top=4, shared_ff=0),
                                                                   2: dict(limit=0.3, scale=0.11)}),
    "no feed-forward": dict(seed=5, mlp=False, streams=2),
    "many heads": dict(seed=6, heads=(20,), dim=8, rot_dim=4, vdim=8, kv_rank=24),
}
_made = {}


def model_of(name, dtype, **engine):
    """Configuration, weights and engine (models are built once per name and dtype, engines per call)."""
    if (name, dtype) not in _made:
        cfg, W = O.random_model(**MODELS[name])
        _made[name, dtype] = cfg, W, GinisunModel(GinisunConfig.from_dict(cfg), {k: torch.tensor(v) for k, v in W.items()}, "cuda", dtype)
    cfg, W, m = _made[name, dtype]
    engine.setdefault("max_tokens", 1024)
    eng = ServingEngine(m, **engine)
    np.random.default_rng(0).shuffle(eng.pool.free)
    return cfg, W, eng


_refs = {}


def reference(name, cfg, W, tokens):
    key = (name, tuple(tokens))
    if key not in _refs:
        _refs[key] = O.forward(cfg, W, list(tokens))
    return _refs[key]


def prompt(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


LOGIT_TOL = {F32: 2e-5, BF16: 6e-2}


def close(got, want, dtype, frac=0.0):
    """f32: every position; bf16: all but a few (a token near the border between two experts may take the other one)."""
    g, w = got.double().cpu().numpy(), np.asarray(want)
    assert g.shape == w.shape and np.isfinite(g).all()
    e = np.sqrt(((g - w) ** 2).mean(-1)) / np.sqrt((w ** 2).mean())
    assert (e > LOGIT_TOL[dtype]).mean() <= (0.0 if dtype == F32 else max(0.1, frac)), np.sort(e)[-5:]
    assert np.median(e) < LOGIT_TOL[dtype] / 2


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", MODELS)
def test_whole_prompts_and_residuals(name, dtype):
    cfg, W, eng = model_of(name, dtype)
    toks = prompt(cfg, 90, 1)
    taps, trace = [], []
    got = eng.step([StepEntry("a", toks, range(90))], ["a"], taps=taps)
    want = O.forward(cfg, W, toks, trace)
    close(got, want, dtype)
    for t, r in zip(taps, trace):
        assert np.median(np.abs(t.double().cpu().numpy() - r)) / np.sqrt((r ** 2).mean()) < (2e-6 if dtype == F32 else 3e-2)
    assert len(taps) == len(cfg["layers"]) and "a" not in eng and eng.pool.num_free() == len(eng.pool.pages)
    close(eng.step([StepEntry("b", toks, [0, 17, 89])], ["b"]), want[[0, 17, 89]], dtype, 0.34)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["plain", "odd sizes", "layers that differ", "many heads"])
def test_token_by_token_equals_prefill(name, dtype):
    """From the very first token, over several page borders."""
    cfg, W, eng = model_of(name, dtype)
    toks = prompt(cfg, 70, 2)
    got = torch.cat([eng.step([StepEntry("a", [t], [0])]) for t in toks])
    close(got, reference(name, cfg, W, toks), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("size", [2, 7, 16, 33])
def test_portions_of_prompts(size, dtype):
    cfg, W, eng = model_of("layers that differ", dtype)
    toks = prompt(cfg, 75, 3)
    out = []
    for i in range(0, 75, size):
        part = toks[i: i + size]
        out.append(eng.step([StepEntry("a", part, range(len(part)))]))
    close(torch.cat(out), reference("layers that differ", cfg, W, toks), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_batches_equal_each_request_alone_and_pages_are_reused(dtype):
    """Unequal requests start together and decode together, shorter ones end earlier; a second set then runs on the freed pages."""
    cfg, W, eng = model_of("plain", dtype, max_tokens=400, max_sequences=6)
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
        assert eng.pool.num_free() == len(eng.pool.pages)
        for k, (p, n) in lens.items():
            close(torch.stack(got[k]), reference("plain", cfg, W, toks[k])[p - 1: p + n], dtype, 0.2)


def test_prompts_join_running_sequences_and_large_decode_batches():
    """One step that holds a prompt, a portion and single tokens; then twenty sequences decoding in one step."""
    cfg, W, eng = model_of("plain", BF16, max_tokens=1200)
    toks = {i: prompt(cfg, 30, 50 + i) for i in range(20)}
    eng.step([StepEntry(0, toks[0][:29]), StepEntry(1, toks[1][:10])])
    got = eng.step([StepEntry(0, toks[0][29:], [0]), StepEntry(1, toks[1][10:29], [18]), StepEntry(2, toks[2][:29], [0, 28])])
    want = [reference("plain", cfg, W, toks[0])[29], reference("plain", cfg, W, toks[1])[28], *reference("plain", cfg, W, toks[2])[[0, 28]]]
    close(got, np.stack(want), BF16, 0.25)
    eng.release(0)
    eng.step([StepEntry(0, toks[0][:29])])
    eng.step([StepEntry(i, toks[i][:29]) for i in range(3, 20)])
    got = eng.step([StepEntry(i, [toks[i][29]], [0]) for i in range(20)])
    close(got, np.stack([reference("plain", cfg, W, toks[i])[29] for i in range(20)]), BF16, 0.15)


def test_captured_decode_equals_plain_launches():
    cfg, W, a = model_of("layers that differ", BF16)
    _, _, b = model_of("layers that differ", BF16, use_graph=False)
    toks = prompt(cfg, 40, 6)
    for eng in (a, b):
        eng.step([StepEntry("s", toks[:5])])
    for t in toks[5:]:
        x, y = a.step([StepEntry("s", [t], [0])]), b.step([StepEntry("s", [t], [0])])
        assert torch.equal(x, y)


def test_long_decoding_over_many_pages():
    cfg, W, eng = model_of("one stream, top one", BF16, max_tokens=400)
    toks = prompt(cfg, 330, 8)
    got = [eng.step([StepEntry("s", toks[:3], [0, 1, 2])])] + [eng.step([StepEntry("s", [t], [0])]) for t in toks[3:]]
    close(torch.cat(got), reference("one stream, top one", cfg, W, toks), BF16)


# -- generation ------------------------------------------------------------------------------------------------------------------------
def test_greedy_generation_through_the_scheduler():
    """f32 against the plain evaluation; bf16 decoding feeds its tokens back on the device and agrees with its own step-by-step run. More requests than
    fit at once, prompts cut into portions."""
    cfg, W, eng = model_of("plain", F32, max_tokens=160, max_sequences=3, prefill_chunk=11)
    prompts = [prompt(cfg, n, 70 + n) for n in (5, 30, 1, 17, 24)]
    out = eng.generate(prompts, GenerationConfig(max_new_tokens=7))
    assert out == [O.greedy(cfg, W, p, 7) for p in prompts]
    assert eng.pool.num_free() == len(eng.pool.pages)
    stop = out[0][3]
    cut = eng.generate(prompts[:1], GenerationConfig(max_new_tokens=7, eos_token_id=stop))
    assert cut[0] == out[0][: out[0].index(stop) + 1]
    _, _, fast = model_of("plain", BF16, max_tokens=400)
    got = fast.generate(prompts, GenerationConfig(max_new_tokens=20))
    for p, o in zip(prompts, got):
        seq, logits = list(p), fast.step([StepEntry("x", p, [len(p) - 1])])
        for t in o:
            top = torch.topk(logits[0], 2)
            assert t == int(top.indices[0]) or float(top.values[0] - logits[0, t]) < 0.05 * float(logits[0].std())
            logits = fast.step([StepEntry("x", [t], [0])])
        fast.release("x")
    fast.check()


def test_sampling_beam_and_speculative_decoding_over_the_engine():
    cfg, W, eng = model_of("plain", F32, max_tokens=900)
    p = prompt(cfg, 9, 90)
    want = O.greedy(cfg, W, p, 6)
    m = eng.as_cached_model()
    ids = torch.tensor([p], device="cuda")
    assert generate(m, m.new_cache, ids, GenerationConfig(max_new_tokens=6))[0, 9:].tolist() == want
    seen = []
    assert generate_with_streamer(m, p, GenerationConfig.greedy(6), lambda t: seen.append(t) or True) == want and seen == want
    beam = beam_search(m, m.new_cache, ids, GenerationConfig(max_new_tokens=6, num_beams=3))

    def score(seq):
        lp = torch.log_softmax(torch.tensor(O.forward(cfg, W, seq[:-1])), -1)
        return float(sum(lp[i, seq[i + 1]] for i in range(8, len(seq) - 1)))
    assert score(beam[0].tolist()) >= score(p + want) - 1e-4
    spec, stats = speculative_generate(m, m.new_cache, m, m.new_cache, ids, SpecDecodeConfig(3, 6))
    assert spec[0, 9:].tolist() == want and stats.acceptance_rate() == 1.0
    c = GenerationConfig(max_new_tokens=5, seed=3).with_temperature(0.9).with_top_k(8)
    one, two = eng.generate([p, p[:4]], c), eng.generate([p], c)
    assert one[0] == two[0] and len(one[1]) == 5                          # a request's draws do not depend on its batch
    import gc
    gc.collect()
    assert eng.pool.num_free() == len(eng.pool.pages)


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
        got = np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        close(torch.tensor(got), want[rows], F32)
    assert not (out / "1.f32").exists()


def test_random_weights_and_limits_of_the_engine():
    cfg = GinisunConfig.uniform(1, 64, 32, 2, 16, 8, 16, 16, 3, 1, 24, 16, streams=2)
    W = RandomGinisunWeights(cfg)
    assert set(W.keys()) == set(cfg.tensor_shapes()) and W["l0.hc1.mix"].shape == (2, 2)
    eng = ServingEngine(GinisunModel(cfg, W), max_tokens=32, max_sequences=2)
    from ferrotorch_b200.errors import InvalidArgument
    for bad in ([StepEntry("a", [])], [StepEntry("a", [64])], [StepEntry("a", [1], [1])], [StepEntry("a", [1]), StepEntry("a", [2])], [StepEntry("a", [1] * 33)]):
        with pytest.raises(InvalidArgument):
            eng.step(bad)
    assert eng.pool.num_free() == len(eng.pool.pages) and "a" not in eng
    with pytest.raises(InvalidArgument):
        GinisunModel(cfg, {k: W[k] for k in W.keys() if k != "l0.mix.uk"})
    with pytest.raises(InvalidArgument):
        GinisunModel(cfg, W, dtype=torch.float16)
