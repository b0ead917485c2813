"""Host side of the Ginisun decoder and of the serving engine: configuration, registry, weight packing, the paged row cache, batch tables, the scheduler's
decisions and the trace replay program."""
import io
import json

import numpy as np
import pytest
import torch

import ginisun_oracle as O
from ferrotorch_b200 import _lib, models
from ferrotorch_b200.errors import InvalidArgument
from ferrotorch_b200.models import (Architecture, CachedEngineModel, CachedLlama, CachedModelEngine, DecodeState, EngineCache, ExpertConfig, GenerationConfig,
                                    GinisunConfig, GinisunLayer, GinisunModel, LatentMixerConfig, LlamaConfig, MoeConfig, RowBatch, Scheduler, ServingEngine, StepEntry,
                                    architecture_of, architectures, load_checkpoint_weights, load_engine, load_model_config, register_architecture)
from ferrotorch_b200.models.llama_infer import random_hf_weights
from ferrotorch_b200.nn import PagedRowCache, PagePool
from ferrotorch_b200.ops import LatentDims, LatentWeights, interleave_gate_up, rotary_pair_tables
from ferrotorch_b200.ops import gated_act, latent_attention_decode, latent_attention_rows  # noqa: F401  (device operators, exercised by the GPU tests)


def test_configuration_reads_every_size_of_every_layer():
    cfg, W = O.random_model(3, heads=(2, 5, 1), overrides={0: dict(mlp=False), 1: dict(dim=24, rot_dim=4, vdim=10, kv_rank=20, experts=7, top=3, ff=9, shared_ff=0, base=77.0)})
    c = GinisunConfig.from_dict(cfg)
    assert {k: tuple(v.shape) for k, v in W.items()} == c.tensor_shapes()
    assert c.layers[0].mlp is None and "l0.norm2" not in W and "l0.hc2.in" not in W
    assert c.layers[1] == GinisunLayer(LatentMixerConfig(5, 24, 4, 10, 20, 28 ** -0.5, 77.0), MoeConfig(7, 3, ExpertConfig(9, 1.25), None))
    assert c.layers[2].mlp.shared == ExpertConfig(40, 0.75) and c.vocab_size == 96
    again = GinisunConfig.from_dict(json.loads(json.dumps(c.to_dict())))
    assert again == c


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4),
                                    lambda c: c["layers"][1]["mlp"]["router"].update(top=6), lambda c: c["layers"][1]["mlp"].update(kind="dense"),
                                    lambda c: c.update(streams=17), lambda c: c.update(layers=[]), lambda c: c["layers"][0]["mixer"].update(scale=0.0),
                                    lambda c: c["layers"][0]["mixer"].update(heads=0)])
def test_configuration_refuses_what_it_cannot_run(change):
    cfg, _ = O.random_model(1)
    change(cfg)
    with pytest.raises(InvalidArgument):
        GinisunConfig.from_dict(cfg)


def test_absent_limit_means_no_limit_and_the_model_needs_a_device():
    assert ExpertConfig.from_dict({"ff": 3}).limit == float("inf") and ExpertConfig(3).to_dict()["limit"] is None
    cfg, W = O.random_model(1)
    with pytest.raises(InvalidArgument):
        GinisunModel(GinisunConfig.from_dict(cfg), W, device="cpu")


def test_registry_finds_the_architecture(tmp_path):
    cfg, W = O.random_model(1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    from ferrotorch_b200.serialize import save_safetensors, save_safetensors_sharded
    state = {k: torch.tensor(v).to(torch.bfloat16) for k, v in W.items()}
    save_safetensors(state, tmp_path / "model.safetensors")
    arch, c = load_model_config(tmp_path)
    assert arch.name == "Ginisun" and isinstance(c, GinisunConfig)
    one = load_checkpoint_weights(tmp_path)
    (tmp_path / "model.safetensors").unlink()
    save_safetensors_sharded(state, tmp_path, max_shard_bytes=20000)
    two = load_checkpoint_weights(tmp_path)
    assert one.keys() == two.keys() == state.keys() and all(torch.equal(one[k], two[k]) for k in one)
    assert architecture_of({"model_type": "llama"}) is architecture_of({"architectures": ["LlamaForCausalLM"]})
    with pytest.raises(InvalidArgument):
        architecture_of({"architecture": "nothing"})
    register_architecture(Architecture("Throwaway", dict, lambda *a: a))
    assert "Throwaway" in architectures() and architecture_of({"architecture": "throwaway"}).name == "Throwaway"
    models.registry._ARCHITECTURES.pop("throwaway")


def test_packed_weights_keep_every_row_where_the_kernels_look():
    g, u = torch.arange(11.0)[:, None] * torch.ones(1, 5) + 100, torch.arange(11.0)[:, None] * torch.ones(1, 5) + 200
    w = interleave_gate_up(g, u, 32)
    assert w.shape == (32, 32) and w[:8, 0].tolist() == list(range(100, 108)) and w[8:16, 0].tolist() == list(range(200, 208))
    assert w[16:24, 0].tolist() == [108, 109, 110, 0, 0, 0, 0, 0] and w[24:27, 0].tolist() == [208, 209, 210] and float(w[:, 5:].abs().sum()) == 0
    D = LatentDims(3, 10, 6, 7, 20, 0.3, 1e-5)
    assert (D.dim8, D.rot8, D.v8, D.rank8, D.r16, D.row, D.q_cols, D.proj_cols) == (16, 8, 8, 24, 32, 48, 72, 104)
    rng = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=rng)
    q, dkv, uk, uv, o = r(48, 9), r(26, 9), r(30, 20), r(21, 20), r(9, 21)
    p = LatentWeights.pack(D, q, dkv, r(20), uk, uv, o, "cpu", torch.float32)
    assert torch.equal(p.proj[24 + 16: 24 + 22], q[16 + 10: 32]) and torch.equal(p.proj[48: 58], q[32: 42]) and float(p.proj[10:16].abs().sum()) == 0
    assert torch.equal(p.proj[72: 92], dkv[:20]) and torch.equal(p.proj[96: 102], dkv[20:])
    assert torch.equal(p.ukv[16: 26, :20], uk[10: 20]) and torch.equal(p.uv[8: 15, :20], uv[7: 14]) and torch.equal(p.out[:, 16: 23], o[:, 14: 21])
    assert p.ukv.shape[0] >= 3 * (16 + 8) + 16 and p.ukv.stride(0) % 32 == 0


def test_flash_tile_sizes_agree_with_the_kernel_library():
    for d in (8, 64, 65, 128, 192, 256, 512):
        for dr in (2, 64, 96):
            for dv in (8, 64, 100, 128, 192, 256, 300):
                assert LatentDims(2, d, dr, dv, 64, 1.0, 1e-5).flash_tile() == _lib.kernels().ft_latent_flash_tile(d, dr, dv), (d, dr, dv)


def test_neighbouring_pairs_turn_by_their_own_frequency():
    cos, sin = rotary_pair_tables(50, 6, 300.0, "cpu")
    x = np.random.default_rng(0).standard_normal((50, 6))
    want = O.rotate_pairs(x, np.arange(50), 300.0)
    c, s = cos.double().numpy(), sin.double().numpy()
    got = np.stack([x[:, 0::2] * c - x[:, 1::2] * s, x[:, 1::2] * c + x[:, 0::2] * s], -1).reshape(50, 6)
    assert np.abs(got - want).max() < 1e-6 and np.allclose((got ** 2).sum(-1), (x ** 2).sum(-1))


# -- cache -----------------------------------------------------------------------------------------------------------------------------
def test_row_cache_pages_are_shared_copied_freed_and_reused():
    pool = PagePool(6, 4)
    c = PagedRowCache(pool, [3, 5])
    c.add_sequence("a")
    with pytest.raises(InvalidArgument):
        c.add_sequence("a")
    assert c.pages_for("a", 6) == 2
    c.reserve("a", 6)
    for p, s in enumerate(c.slots("a", 0, 6)):
        for r in c.rows:
            r.flatten(0, 1)[s] = p + 1
    c.lengths["a"] = 6
    c.fork("a", "b")
    assert pool.num_free() == 4 and c.tables["a"] == c.tables["b"]
    c.reserve("b", 7)                                    # b writes position 6: its half-full page becomes its own
    assert c.tables["a"][0] == c.tables["b"][0] and c.tables["a"][1] != c.tables["b"][1] and pool.num_free() == 3
    for layer in (0, 1):
        assert torch.equal(c.gather(layer, "a"), c.gather(layer, "b")) and c.gather(layer, "b")[:, 0].tolist() == [1, 2, 3, 4, 5, 6]
    shared = c.tables["a"][0]
    c.free_sequence("a")
    assert shared not in pool.free and pool.num_free() == 4
    c.truncate("b", 3)
    assert c.lengths["b"] == 3 and len(c.tables["b"]) == 1 and pool.num_free() == 5
    c.add_sequence("c")
    c.reserve("c", 20)
    assert pool.num_free() == 0 and shared not in c.tables["c"]
    t = c.block_table(["c", "b"], 6)
    assert t[0, :5].tolist() == c.tables["c"] and t[0, 5] == -1 and t[1].tolist() == [shared, -1, -1, -1, -1, -1]
    with pytest.raises(InvalidArgument):
        c.reserve("b", 5)


def test_batch_tables():
    c = PagedRowCache(PagePool(20, 16), [4])
    for k, n in (("x", 0), ("y", 18)):
        c.add_sequence(k)
        c.reserve(k, 60)
        c.lengths[k] = n
    b = RowBatch([StepEntry("x", [5, 6, 7], [2]), StepEntry("y", list(range(40)), [0, 39])], c, "cpu", 8)
    assert b.rows == 43 and b.ctx_total == 3 + 58 and not b.single
    assert b.positions.tolist() == [0, 1, 2] + list(range(18, 58)) and b.seq_of.tolist() == [0] * 3 + [1] * 40
    assert b.slots.tolist() == c.slots("x", 0, 3) + c.slots("y", 18, 40)
    assert b.ctx_rows.tolist() == [0, 1, 2] + list(range(21, 61)) and b.past_slots.tolist() == c.slots("y", 0, 18) and b.past_rows.tolist() == list(range(3, 21))
    assert b.want.tolist() == [2, 3, 42]
    small = LatentDims(1, 16, 16, 16, 16, 1.0, 1e-5)
    assert small.flash_tile() == 128 and b.tiles_for(small).tolist() == [[3, 40, 18, 3], [0, 3, 0, 0]]
    c.lengths["y"] = 0
    b = RowBatch([StepEntry("y", [1] * 60)], c, "cpu", 8)
    assert b.past_slots is None and b.want is None
    assert b.tiles_for(LatentDims(1, 500, 16, 16, 16, 1.0, 1e-5)) is None
    s = DecodeState("cpu", 8)
    s.load([4, 9], [17, 0], c.block_table(["y", "x"], 8))
    assert s.positions[:2].tolist() == [17, 0] and s.seq_lens[:2].tolist() == [18, 1] and s.tokens[:2].tolist() == [4, 9]
    assert s.block_table[0].tolist() == c.block_table(["y"], 8)[0].tolist() and s.block_table[1, 0] == c.tables["x"][0]


# -- engine and scheduler on a stand-in model -------------------------------------------------------------------------------------------
class CountingModel:
    """Next token = (sum of all tokens of the sequence) mod vocab, remembered through the engine's page cache only."""
    vocab, dtype, device, cache_rows, cfg = 50, torch.float32, "cpu", [1], LlamaConfig.tiny(vocab=50)

    def __init__(self):
        self.steps = []

    def prepare(self, n):
        self.positions = n

    def decode_supported(self):
        return False

    def forward_rows(self, batch, cache, taps=None):
        rows = cache.rows[0].view(-1)
        rows[batch.slots.long()] = batch.ids.float()
        self.steps.append((batch.rows, batch.block_table.shape[0], batch.single))
        logits = torch.zeros(batch.rows, self.vocab)
        for i in range(batch.rows):
            t = batch.block_table[batch.seq_of[i]].long()
            n = int(batch.positions[i]) + 1
            idx = (t[:, None] * 16 + torch.arange(16)).view(-1)[:n]
            logits[i, int(rows[idx].sum()) % self.vocab] = 1.0
        return None if batch.want is None else logits[batch.want]


def _expected(p, n):
    seq = list(p)
    for _ in range(n):
        seq.append(sum(seq) % 50)
    return seq[len(p):]


def test_scheduler_admits_cuts_and_finishes_requests():
    m = CountingModel()
    eng = ServingEngine(m, max_tokens=96, max_sequences=3, prefill_chunk=10)
    assert m.positions == 96
    prompts = [[1, 2, 3], list(range(25)), [7], [9] * 12, [3, 1]]
    assert eng.generate(prompts, GenerationConfig(max_new_tokens=5)) == [_expected(p, 5) for p in prompts]
    assert max(s[0] for s in m.steps) <= 10 and max(s[1] for s in m.steps) <= 3 and eng.pool.num_free() == len(eng.pool.pages)
    seen = []
    stop = _expected(prompts[0], 5)[2]
    out = eng.generate(prompts[:2], GenerationConfig(max_new_tokens=5, eos_token_id=stop), streamer=lambda i, t: seen.append((i, t)))
    assert out[0] == _expected(prompts[0], 5)[:3] and [t for i, t in seen if i == 1] == out[1]
    s = Scheduler(eng, GenerationConfig(max_new_tokens=80))
    with pytest.raises(InvalidArgument):
        s.submit(list(range(20)))                          # would not fit to its last token
    with pytest.raises(InvalidArgument):
        s.submit([])
    with pytest.raises(InvalidArgument):
        Scheduler(eng, GenerationConfig(num_beams=2))
    assert eng.generate([[1]], GenerationConfig(max_new_tokens=0)) == [[]]


def test_step_order_release_and_cached_model_interface():
    m = CountingModel()
    eng = ServingEngine(m, max_tokens=64, max_sequences=4)
    out = eng.step([StepEntry("a", [1, 2, 3], [2, 0]), StepEntry("b", [4], [0])])
    assert out.argmax(-1).tolist() == [6, 1, 4] and eng.length("a") == 3 and "b" in eng
    assert eng.step([StepEntry("a", [10])], ["b"]) is None and "b" not in eng
    assert eng.step([StepEntry("a", [1], [0])], ["a"]).argmax(-1).tolist() == [17] and eng.pool.num_free() == len(eng.pool.pages)
    cm = eng.as_cached_model()
    assert isinstance(cm, CachedEngineModel)
    c = cm.new_cache()
    assert isinstance(c, EngineCache) and c.len() == 0
    assert cm(torch.tensor([[5, 6]]), c).argmax(-1).tolist() == [[5, 11]] and c.len() == 2
    c.expand(3)
    assert cm(torch.tensor([[1], [2], [3]]), c).argmax(-1).flatten().tolist() == [12, 13, 14]
    c.reorder(torch.tensor([2, 2, 0]))
    assert cm(torch.tensor([[0], [1], [0]]), c).argmax(-1).flatten().tolist() == [14, 15, 12]
    c.truncate(2)
    assert c.len() == 2 and cm(torch.tensor([[0], [0], [0]]), c).argmax(-1).flatten().tolist() == [11] * 3
    del c
    import gc
    gc.collect()
    assert eng.pool.num_free() == len(eng.pool.pages)


def test_trace_replay_of_a_llama_checkpoint_on_the_host(tmp_path):
    """The program chooses the engine by config.json; here the cached Llama decoder."""
    from ferrotorch_b200.models import trace
    from ferrotorch_b200.serialize import save_safetensors
    cfg = LlamaConfig(vocab_size=40, hidden_size=32, intermediate_size=48, num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, max_position_embeddings=64)
    W = random_hf_weights(cfg, "cpu", 1, 0.2)
    (tmp_path / "config.json").write_text(json.dumps({**cfg.to_dict(), "model_type": "llama"}))
    save_safetensors(W, tmp_path / "model.safetensors")
    eng = load_engine(tmp_path, "cpu", torch.float32, 64)
    assert isinstance(eng, CachedModelEngine)
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": [1, 2, 3], "want": [0, 2]}, {"id": "q", "tokens": [4], "want": [0]}], "end": ["q"]},
             {"step": 1, "entries": [{"id": "p", "tokens": [7], "want": []}], "end": []}, {"step": 2, "entries": [{"id": "p", "tokens": [8], "want": [0]}], "end": ["p"]}]
    said = io.StringIO()
    assert trace.replay(eng, [json.dumps(s) + "\n" for s in steps] + ["\n"], tmp_path, said) == 3
    assert said.getvalue() == "done 0\ndone 1\ndone 2\n" and not (tmp_path / "1.f32").exists() and "p" not in eng
    m = CachedLlama(cfg, {k: v.float() for k, v in W.items()})
    whole = m(torch.tensor([[1, 2, 3, 7, 8]]), m.new_cache())[0]
    first = np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(3, 40)
    assert np.abs(first[:2] - whole[[0, 2]].numpy()).max() < 1e-5
    assert np.abs(np.fromfile(tmp_path / "2.f32", dtype="<f4") - whole[4].numpy()).max() < 1e-5
    from ferrotorch_b200.models import generate
    want = generate(m, m.new_cache, torch.tensor([[1, 2, 3]]), GenerationConfig(max_new_tokens=4))[0, 3:].tolist()
    assert eng.generate([[1, 2, 3]], GenerationConfig(max_new_tokens=4)) == [want]
