"""Host side of the Pufevik decoder and of recurrent state in the serving engine: configuration, registry, weight packing, state slots, batch tables, and the engine and
scheduler on a stand-in model whose memory is a state alone."""
import json

import numpy as np
import pytest
import torch

import pufevik_oracle as O
from ferrotorch_b200 import _build, _lib
from ferrotorch_b200.errors import InvalidArgument, ShapeMismatch
from ferrotorch_b200.models import (AttentionConfig, DecodeState, GenerationConfig, LlamaConfig, MemoryConfig, ParallelConfig, PufevikConfig, PufevikLayer, PufevikModel, RowBatch,
                                    ServingEngine, StepEntry, architectures, checked_weights, load_model_config, registry)
from ferrotorch_b200.nn import PagedRowCache, PagePool, StateSlots
from ferrotorch_b200.ops import DenseGatedWeights, GqaDims, GqaWeights, MemoryDims, pack_head_columns, pack_head_rows, pack_head_vector
from ferrotorch_b200.ops import dense_gated_rows, gqa_attention_decode, matrix_memory_decode, residual_update  # noqa: F401  (device operators, exercised by the GPU tests)


def test_configuration_reads_every_size_of_every_layer():
    cfg, W = O.random_model(3, kinds="apa", overrides={0: dict(ff=0, v_mix=False, rot=0), 1: dict(window=77, cap=3.5, left_scale=0.25, right_scale=1.75, mem_heads=5, kv_heads=1, base=9.0)})
    c = PufevikConfig.from_dict(cfg)
    assert {k: tuple(v.shape) for k, v in W.items()} == c.tensor_shapes()
    assert c.layers[0] == PufevikLayer(AttentionConfig(4, 2, 16, 24, 0.25, 0, 10000.0), 0) and "l0.norm2" not in W and "l0.mix.vmix" not in W
    assert c.layers[1] == PufevikLayer(ParallelConfig(AttentionConfig(4, 1, 16, 24, 0.25, 8, 9.0, 77), MemoryConfig(5, 16, 16, 3.5), 0.25, 1.75), 72)
    assert c.layers[2].mixer.v_mix and c.mixing_layers == [2] and c.optional_tensors == ["l0.mix.vmix", "l2.mix.vmix"] and c.vocab_size == 90 and c.embedding_scale == 3.0
    assert PufevikConfig.from_dict(json.loads(json.dumps(c.to_dict()))) == c


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7),
                                    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), lambda c: c["layers"][1]["mixer"].update(heads=3),
                                    lambda c: c["layers"][1]["mlp"].update(kind="moe"), lambda c: c["layers"][0]["mlp"].update(ff=0), lambda c: c.update(layers=[]),
                                    lambda c: c["layers"][1]["mixer"].update(scale=0.0), lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=0),
                                    lambda c: c["layers"][0]["mixer"]["left"].update(v_mix=True), lambda c: c["layers"][1]["mixer"].update(mask=dict(size=4)),
                                    lambda c: c["layers"][2]["mixer"].update(vdim=8)])
def test_configuration_refuses_what_it_cannot_run(change):
    cfg, _ = O.random_model(1, kinds="paa")
    change(cfg)
    with pytest.raises(InvalidArgument):
        PufevikConfig.from_dict(cfg)


def test_registry_weights_and_device(tmp_path):
    cfg, W = O.random_model(1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    arch, c = load_model_config(tmp_path)
    assert arch.name == "Pufevik" and isinstance(c, PufevikConfig) and {"Pufevik", "Ginisun"} <= set(architectures())
    with pytest.raises(InvalidArgument):
        PufevikModel(c, {k: torch.tensor(v) for k, v in W.items()}, device="cpu")
    shapes = {"a": (2, 3), "b": ()}
    get = checked_weights("x", shapes, {"a": torch.zeros(2, 3), "c": torch.zeros(1)}, "cpu", optional=("b", "c"))
    assert get("a").shape == (2, 3)
    for bad in ({"b": torch.zeros(())}, {"a": torch.zeros(2, 3), "b": torch.zeros(()), "d": torch.zeros(1)}):
        with pytest.raises(InvalidArgument):
            checked_weights("x", shapes, bad, "cpu")
    with pytest.raises(ShapeMismatch):
        checked_weights("x", {"a": (3, 2)}, {"a": torch.zeros(2, 3)}, "cpu")("a")


def test_the_reference_agrees_with_itself():
    """The plain evaluation's recurrence against the closed form of a stretch, and its attention against one query at a time."""
    rng = np.random.default_rng(0)
    q, k, v, i = rng.standard_normal((9, 4)), rng.standard_normal((9, 4)), rng.standard_normal((9, 3)), rng.standard_normal(9)
    f = -np.logaddexp(0.0, -rng.standard_normal(9))
    got, (S, n, m) = O.matrix_memory(q, k, v, i, f)
    F = np.cumsum(f)
    for t in range(9):
        top = F[t] + max(0.0, (i[: t + 1] - F[: t + 1]).max())
        w = np.exp(F[t] - F[: t + 1] + i[: t + 1] - top)
        assert np.allclose(got[t], (w * (k[: t + 1] @ q[t])) @ v[: t + 1] / (max(abs((w * (k[: t + 1] @ q[t])).sum()), np.exp(-top)) + 1e-6))
    assert np.isclose(m, top) and np.allclose(S, (w[:, None] * k).T @ v) and np.allclose(n, w @ k)
    a = O.attend(q[:, None], k[:, None], v[:, None], 0.7, window=3, sink=np.array([0.4]))
    for t in range(9):
        s = np.exp(0.7 * k[max(0, t - 2): t + 1] @ q[t])
        assert np.allclose(a[t, 0], s @ v[max(0, t - 2): t + 1] / (s.sum() + np.exp(0.4)))


def test_packed_weights_keep_every_row_where_the_kernels_look():
    w = torch.arange(30.0).reshape(10, 3)
    r = pack_head_rows(w, 2, 5, "cpu", torch.float32)
    assert r.shape == (32, 3) and torch.equal(r[:5], w[:5]) and torch.equal(r[16:21], w[5:]) and float(r[5:16].abs().sum()) == 0
    c = pack_head_columns(w.t(), 2, 5, "cpu", torch.float32)
    assert c.shape == (3, 32) and torch.equal(c[:, 16:21], w[5:].t())
    assert pack_head_vector(torch.arange(1.0, 11), 2, 5, "cpu").nonzero().flatten().tolist() == [0, 1, 2, 3, 4, 16, 17, 18, 19, 20]
    D = GqaDims(6, 2, 20, 40, 8, 0.3, 1e-5, whole_norm=True)
    assert (D.d16, D.v16, D.k_col, D.v_col, D.qkv_cols, D.out_cols, D.row) == (32, 48, 192, 256, 352, 288, 160)
    g = GqaWeights.pack(D, torch.ones(120), torch.ones(40), "cpu")
    assert g.q_norm.shape == (192,) and g.k_norm.shape == (64,) and g.sink is None and float(g.q_norm.sum()) == 120
    M = MemoryDims(3, 20, 40, 5.0, 1e-5)
    assert (M.h8, M.gate_col, M.proj_cols, M.out_cols, M.state_size) == (8, 3 * (64 + 48), 3 * (64 + 96), 144, 3 * (32 * 48 + 32 + 4))
    d = DenseGatedWeights.pack(torch.ones(11, 5), 2 * torch.ones(11, 5), torch.ones(5, 11), "cpu", torch.float32)
    assert d.fp == 16 and d.gu.shape == (32, 5) and d.gu[:, 0].tolist() == [1] * 8 + [2] * 8 + [1] * 3 + [0] * 5 + [2] * 3 + [0] * 5 and d.down.stride(0) % 32 == 0


def test_size_limits_of_the_kernels():
    L = _lib.kernels()
    for heads, kv, d, dv, sub in ((8, 1, 64, 64, 1), (8, 2, 128, 128, 1), (4, 4, 96, 100, 1), (4, 4, 192, 100, 2), (1, 1, 256, 256, 1), (2, 1, 1024, 64, 0), (130, 1, 64, 64, 0)):
        assert L.ft_gqa_flash_subtiles(heads, kv, d, dv, 1) == sub, (heads, kv, d, dv)
        assert GqaDims(heads, kv, d, dv, 0, 1.0, 1e-5).flash_tile() == sub * (128 // (heads // kv))
    assert GqaDims(130, 1, 64, 64, 0, 1.0, 1e-5).decode_supported() and not GqaDims(1, 1, 600, 64, 0, 1.0, 1e-5).decode_supported()
    assert MemoryDims(1, 256, 999, 1.0, 1e-5).walk_supported() and not MemoryDims(1, 272, 16, 1.0, 1e-5).walk_supported()
    assert MemoryDims(1, 1024, 1024, 1.0, 1e-5).decode_supported() and not MemoryDims(1, 16, 1040, 1.0, 1e-5).decode_supported()


@pytest.mark.parametrize("name", ["pufevik", "ginisun"])
def test_a_partial_kernel_library_is_complete(name):
    """The sources that an architecture names link without the rest."""
    import ctypes
    lib = _build.build_kernels_part(f"{name}_test", registry._ARCHITECTURES[name].kernels)
    try:
        h = ctypes.CDLL(str(lib))          # unresolved symbols would show here
        assert h.ft_abi_version() == 1 and hasattr(h, "ft_gemm_bf16_splitk") and not hasattr(h, "ft_layernorm_fwd")
    finally:
        lib.unlink()


# -- state slots and batch tables --------------------------------------------------------------------------------------------------------
def test_state_slots_are_owned_copied_and_reused():
    s = StateSlots(2, [3, 0, 5])
    assert s.data[0].shape == (3, 3) and s.data[1] is None and s.spare == 2
    c = PagedRowCache(PagePool(8, 4), [1], states=s)
    c.add_sequence("a")
    s.data[0][s.slot["a"]], s.data[2][s.slot["a"]] = 7.0, 8.0
    c.reserve("a", 6)
    c.lengths["a"] = 6
    c.fork("a", "b")
    assert s.slot["a"] != s.slot["b"] and s.data[0][s.slot["b"]].tolist() == [7.0] * 3 and s.data[2][s.slot["b"]].tolist() == [8.0] * 5 and s.num_free() == 0
    for add in (lambda: c.add_sequence("c"), lambda: c.fork("a", "c")):
        with pytest.raises(InvalidArgument):
            add()
    assert "c" not in c.tables
    with pytest.raises(InvalidArgument):
        c.truncate("a", 3)
    c.truncate("a", 6)
    c.truncate("a", 0)
    assert c.lengths["a"] == 0
    c.free_sequence("a")
    c.free_sequence("b")
    assert s.num_free() == 2 and not s.slot


def _batch(lens, starts, max_sequences=8):
    s = StateSlots(max_sequences, [4])
    c = PagedRowCache(PagePool(600, 16), [4], states=s)
    for k, (n, st) in enumerate(zip(lens, starts)):
        c.add_sequence(k)
        c.reserve(k, n + st)
        c.lengths[k] = st
    return RowBatch([StepEntry(k, [0] * n) for k, n in enumerate(lens)], c, "cpu", 600), s


def test_query_tiles_cover_every_row_once():
    b, _ = _batch([40, 3, 17], [18, 0, 100])
    t = b.query_tiles(16).tolist()
    assert sorted(t) == sorted([[0, 16, 18, 0], [16, 16, 34, 0], [32, 8, 50, 0], [40, 3, 0, 1], [43, 16, 100, 2], [59, 1, 116, 2]])
    assert t[0] == [59, 1, 116, 2] or t[0] == [43, 16, 100, 2] and b.query_tiles(16) is b.query_tiles(16)


@pytest.mark.parametrize("ctas", [0, 1, 16, 32, 400])
def test_memory_plans_cut_long_stretches_into_chained_segments(ctas):
    lens, starts = [4096, 5, 700], [0, 9, 3]
    b, s = _batch(lens, starts)
    p = b.memory_plan(ctas)
    rows = p.segments.tolist()
    seen, at = [], 0
    for i, (n, st) in enumerate(zip(lens, starts)):
        mine = [r for r in rows if r[3] == i]
        for r in mine:
            assert r[0] == at and r[2] == s.slot[i] and bool(r[4] & 4) == (st == 0)
            at += r[1]
        assert all(r[1] == mine[0][1] and (not ctas or r[1] % 128 == 0) for r in mine[:-1]) and (len(mine) == 1 or mine[0][1] >= 128)
        assert [r[4] & 3 for r in mine] == ([3] if len(mine) == 1 else [0] * (len(mine) - 1) + [2])
        c = p.chains.tolist()[i]
        assert c[1:] == [len(mine), s.slot[i], int(st == 0)]
        if len(mine) > 1:
            assert [r[5] for r in mine] == list(range(c[0], c[0] + len(mine)))
            seen += [r[5] for r in mine]
    assert at == sum(lens) and seen == list(range(p.scratch)) and p.sequences == 3
    assert (p.inner is None) == (p.scratch == 0) and (p.inner is None or p.inner.tolist() == [r for r in rows if not r[4] & 2])
    assert len(rows) == {0: 3, 1: 20, 16: 10, 32: 6, 400: 3}[ctas]


def test_decode_state_carries_slots():
    st = DecodeState("cpu", 4)
    st.load([4, 9], [17, 0], torch.tensor([[3, 5, -1, -1], [2, -1, -1, -1]], dtype=torch.int32), [6, 1])
    assert st.slots[:2].tolist() == [6, 1] and st.positions[:2].tolist() == [17, 0] and st.seq_lens[:2].tolist() == [18, 1] and st.block_table[1, 0] == 2


# -- engine and scheduler on a stand-in model --------------------------------------------------------------------------------------------
class SummingModel:
    """Next token = (3 * state + token) mod vocab, state = running combination of all tokens, kept in the engine's slots only."""
    vocab, dtype, device, cache_rows, state_sizes, cfg = 50, torch.float32, "cpu", [1], [1], LlamaConfig.tiny(vocab=50)

    def prepare(self, n):
        pass

    def decode_supported(self):
        return False

    def forward_rows(self, batch, cache, taps=None):
        plan = batch.memory_plan(0)
        data = cache.states.data[0]
        logits = torch.zeros(batch.rows, self.vocab)
        for r0, n, slot, _, flags, *_ in plan.segments.tolist():
            s = 0 if flags & 4 else int(data[slot])
            for r in range(r0, r0 + n):
                s = (3 * s + int(batch.ids[r])) % 50
                logits[r, s] = 1.0
            data[slot] = s
        return None if batch.want is None else logits[batch.want]


def _expected(p, n):
    s, seq = 0, list(p)
    for t in seq:
        s = (3 * s + t) % 50
    out = []
    for _ in range(n):
        out.append(s)
        s = (3 * s + s) % 50
    return out


def test_recurrent_requests_through_the_scheduler():
    eng = ServingEngine(SummingModel(), max_tokens=96, max_sequences=3, prefill_chunk=10)
    eng.states.data[0].fill_(31)                                    # leftovers of nobody
    prompts = [[1, 2, 3], list(range(25)), [7], [9] * 12, [3, 1]]
    for _ in range(2):
        assert eng.generate(prompts, GenerationConfig(max_new_tokens=5)) == [_expected(p, 5) for p in prompts]
        assert eng.states.num_free() == 3 and eng.pool.num_free() == len(eng.pool.pages) and not eng._fed


def test_steps_forks_and_truncation_of_recurrent_sequences():
    eng = ServingEngine(SummingModel(), max_tokens=64, max_sequences=4)
    assert eng.step([StepEntry("a", [1, 2, 3], [2])]).argmax(-1).tolist() == _expected([1, 2, 3], 1)
    eng.fork("a", "b")
    eng.step([StepEntry("a", [4, 5])])
    assert eng.step([StepEntry("b", [8], [0])]).argmax(-1).tolist() == _expected([1, 2, 3, 8], 1)
    eng.truncate("a", 4)
    assert eng.length("a") == 4 and eng.step([StepEntry("a", [6], [0])], ["a"]).argmax(-1).tolist() == _expected([1, 2, 3, 4, 6], 1)
    eng.truncate("b", 0)
    assert eng.step([StepEntry("b", [2, 2], [1])], ["b"]).argmax(-1).tolist() == _expected([2, 2], 1)
    with pytest.raises(InvalidArgument):
        eng.step([StepEntry(i, [1]) for i in range(5)])
    assert eng.states.num_free() == 4 and not eng._fed
    cm = eng.as_cached_model()
    c = cm.new_cache()
    assert cm(torch.tensor([[5, 6]]), c).argmax(-1)[0, 1] == _expected([5, 6], 1)[0]
    c.expand(2)
    assert cm(torch.tensor([[1], [2]]), c).argmax(-1).flatten().tolist() == [_expected([5, 6, t], 1)[0] for t in (1, 2)]
    c.reorder(torch.tensor([1, 1]))
    c.truncate(2)
    assert c.len() == 2 and cm(torch.tensor([[3], [4]]), c).argmax(-1).flatten().tolist() == [_expected([5, 6, t], 1)[0] for t in (3, 4)]
    del c
    import gc
    gc.collect()
    assert eng.states.num_free() == 4
