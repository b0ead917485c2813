"""Host side of the Vemepel decoder: configuration, registry, weight packing, batch tables, size limits, and the plain reference against closed forms."""
import ctypes
import json
import math

import numpy as np
import pytest
import torch

import vemepel_oracle as O
from ferrotorch_b200 import _build, _lib
from ferrotorch_b200.errors import InvalidArgument, ShapeMismatch
from ferrotorch_b200.models import (DenseConfig, DifferentialConfig, ExpertConfig, GatedLatentConfig, MoeConfig, RandomVemepelWeights, RotaryGatedLatentConfig, RowBatch, StepEntry,
                                    VemepelConfig, VemepelLayer, VemepelModel, architectures, load_model_config, registry)
from ferrotorch_b200.nn import PagedRowCache, PagePool, StateSlots
from ferrotorch_b200.ops import DensePolyWeights, GqaDims, GqaWeights, LatentDims, LatentWeights, MoeWeights, RouteRule, differential_blend
from ferrotorch_b200.ops.gqa_attention import GATE_ELEMENT, GATE_HEAD


def test_configuration_reads_every_size_of_every_layer():
    cfg, W = O.random_model(3, kinds="arala", logit_scale=0.3, overrides={0: dict(mlp="dense", dense_ff=11, chunk=77), 1: dict(mlp=None, base=300.0, scale=0.7), 2: dict(kv_from=0, heads=8, diff=0.1, chunk=0),
                                                                          3: dict(lat_heads=7, kv_rank=5), 4: dict(experts=5, top=4, ff=9)})
    c = VemepelConfig.from_dict(cfg)
    assert {k: tuple(v.shape) for k, v in W.items()} == c.tensor_shapes()
    moe = MoeConfig(8, 3, ExpertConfig(40))
    assert c.layers[0] == VemepelLayer(DifferentialConfig(4, 2, 12, 20, 12 ** -0.5, 0.35, 77), DenseConfig(11)) and c.layers[0].type == "attention"
    assert c.layers[1] == VemepelLayer(RotaryGatedLatentConfig(3, 16, 20, 32, 0.7, 8, 300.0), None) and c.layers[1].type == "latent_attention_2" and "l1.norm2" not in W
    assert c.layers[2] == VemepelLayer(DifferentialConfig(8, 2, 12, 20, 12 ** -0.5, 0.1, 0, 0), moe) and "l2.mix.k" not in W and "l2.mix.lq1" in W and c.source(2) == 0 and c.source(4) == 4
    assert c.layers[3] == VemepelLayer(GatedLatentConfig(7, 16, 20, 5, 0.25), moe) and c.layers[3].type == "latent_attention" and W["l3.mix.g"].shape == (7, 56) and W["l1.mix.g"].shape == (60, 56)
    assert c.layers[4].mlp == MoeConfig(5, 4, ExpertConfig(9)) and W["l4.dwa"].shape == (6,)
    assert c.logit_scale == 0.3 and c.vocab_size == 90 and c.optional_tensors == ["l1.norm2", "l1.norm2b"]
    assert VemepelConfig.from_dict(json.loads(json.dumps(c.to_dict()))) == c
    r = RandomVemepelWeights(c, device="cpu")
    assert all(tuple(r[k].shape) == s and r[k].dtype == torch.bfloat16 for k, s in c.tensor_shapes().items()) and "l0.shift" in r
    p = VemepelConfig.pattern("arlsas", 64, 32, dict(heads=2, kv_heads=1, dim=8, vdim=8, scale=0.3, diff=0.2, mask=dict(size=5)), dict(heads=2, dim=8, vdim=8, kv_rank=8, scale=0.3),
                              dict(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=8, scale=0.3, rot=dict(base=10.0, dims=4)), moe, dense_ff=24)
    assert [p.source(i) for i in range(6)] == [0, 1, 2, 0, 4, 4] and [isinstance(l.mlp, DenseConfig) for l in p.layers] == [True, False] * 3


def _set(i, part, **kw):
    return lambda c: c["layers"][i][part].update(**kw)


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="other"), _set(0, "mixer", heads=3), _set(0, "mixer", dim=0), _set(0, "mixer", mask=dict(size=-4)), _set(0, "mixer", scale=0.0),
                                    _set(1, "mixer", rot_dim=6), _set(1, "mixer", rot_dim=7, rot=dict(base=1e4, dims=7)), _set(1, "mixer", rot=dict(base=-1.0, dims=8)), _set(2, "mixer", kv_rank=0),
                                    _set(3, "mixer", kv_from=1), _set(3, "mixer", kv_from=3), _set(3, "mixer", kv_from=-1), _set(3, "mixer", dim=13), _set(3, "mixer", vdim=21),
                                    _set(3, "mixer", kv_heads=4), _set(0, "mixer", kv_from=3), _set(0, "mlp", kind="other"), lambda c: c["layers"][0]["mlp"]["router"].update(top=9),
                                    lambda c: c["layers"][0]["mlp"]["router"].update(groups=dict(count=4, keep=2)), lambda c: c["layers"][0]["mlp"]["router"].update(scale=2.0),
                                    lambda c: c["layers"][0]["mlp"]["expert"].update(limit=2.0), _set(0, "mlp", shared=dict(ff=8)), _set(4, "mlp", ff=0), lambda c: c.update(layers=[]),
                                    lambda c: c.update(vocab=0)])
def test_configuration_refuses_what_it_cannot_run(change):
    cfg, _ = O.random_model(1, kinds="arlaa", overrides={3: dict(kv_from=0), 4: dict(mlp="dense")})
    VemepelConfig.from_dict(cfg)
    change(cfg)
    with pytest.raises(InvalidArgument):
        VemepelConfig.from_dict(cfg)


def test_keys_are_borrowed_from_their_owner_only():
    cfg, _ = O.random_model(1, kinds="aaa", overrides={1: dict(kv_from=0), 2: dict(kv_from=1)})
    with pytest.raises(InvalidArgument):
        VemepelConfig.from_dict(cfg)


def test_registry_weights_and_device(tmp_path):
    cfg, W = O.random_model(1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    arch, c = load_model_config(tmp_path)
    assert arch.name == "Vemepel" and isinstance(c, VemepelConfig) and "Vemepel" in architectures()
    with pytest.raises(InvalidArgument):
        VemepelModel(c, {k: torch.tensor(v) for k, v in W.items()}, device="cpu")
    with pytest.raises(ShapeMismatch):
        registry.checked_weights("Vemepel", c.tensor_shapes(), {**{k: torch.tensor(v) for k, v in W.items()}, "l0.shift": torch.zeros(3)}, "cpu")("l0.shift")


def test_a_partial_kernel_library_is_complete():
    """The sources that the architecture names link without the rest."""
    lib = _build.build_kernels_part("vemepel_test", registry._ARCHITECTURES["vemepel"].kernels)
    try:
        h = ctypes.CDLL(str(lib))          # unresolved symbols would show here
        assert h.ft_abi_version() == 1 and all(hasattr(h, n) for n in ("ft_gqa_differential", "ft_latent_gate", "ft_moe_topk", "ft_depth_update", "ft_token_shift", "ft_poly_norm")) and not hasattr(h, "ft_ssm_walk")
    finally:
        lib.unlink()


def test_the_reference_agrees_with_closed_forms():
    rng = np.random.default_rng(0)
    # masks by hand
    see = O.visible(7, 3)
    assert [[j for j in range(7) if see[i, j]] for i in (0, 2, 3, 5, 6)] == [[0], [0, 1, 2], [3], [3, 4, 5], [6]]
    assert O.visible(7).sum() == 28
    # equal maps leave 1 - factor of the values, whose size the norm takes away; opposite factors turn the sign
    q, k, v = rng.standard_normal((5, 2, 1, 3)).repeat(2, 2), rng.standard_normal((5, 1, 1, 3)).repeat(2, 2), rng.standard_normal((5, 1, 6))
    a, b = (O.differential(q, k, v, 0.5, O.visible(5), f, 0.25, 0.0) for f in (0.4, 2.0))
    assert np.allclose(a, -b) and np.allclose((a * a).mean(-1), 0.75 ** 2) and np.allclose(a[0, 0], 0.75 * O.rms(v[0, 0], 0.0))
    assert math.isclose(O.blend(np.zeros(3), np.ones(3), np.ones(3), np.zeros(3), 0.3), 0.3) and math.isclose(O.blend(np.ones(2), np.ones(2), np.zeros(2), np.zeros(2), 0.0), math.exp(2) - 1)
    # rotation keeps lengths and depends on distances only; the first pair turns one radian per position
    x, y = rng.standard_normal((2, 1, 1, 6))
    p, r = (O.rotate_pairs(x, [t], 4, 30.0) * O.rotate_pairs(y, [t - 3], 4, 30.0) for t in (3, 40))
    assert np.isclose(p[..., :4].sum(), r[..., :4].sum()) and np.allclose(O.rotate_pairs(x, [9], 4, 30.0)[..., 4:], x[..., 4:])
    assert np.allclose(O.rotate_pairs(np.array([[[1.0, 0.0]]]), [2], 2, 50.0), [[[math.cos(2), math.sin(2)]]])
    # shift, average, activation
    h = np.arange(6.0).reshape(3, 2)
    assert np.allclose(O.token_shift(h, np.array([0.0, 1.0])), [[0, 0], [2, 1], [4, 3]]) and np.allclose(O.depth_average([h, 2 * h], [1.0, -0.25]), 0.5 * h)
    assert np.allclose(O.poly_norm(np.full((1, 4), 3.0), [1.0, 2.0, 3.0, 4.0], 0.0), 10.0) and np.allclose(O.poly_norm(np.full((1, 4), -3.0), [1.0, 2.0, 3.0, 4.0], 0.0), 2.0)
    e, w = O.route(np.array([0.0, math.log(3.0), -5.0, 0.0]), 2)
    assert e == [1, 0] and np.allclose(w, [0.75, 0.25])


def test_packed_weights_keep_every_row_where_the_kernels_look():
    D = GqaDims(2, 1, 5, 7, 0, 1.0, 1e-5, norm=False, maps=2, chunk=9, diff=0.4)
    assert (D.k_col, D.v_col, D.qkv_cols, D.out_cols, D.row, D.turned) == (64, 96, 112, 32, 48, False)
    S = GqaDims(2, 1, 5, 7, 0, 1.0, 1e-5, norm=False, maps=2, own=False)
    assert S.qkv_cols == 64 and S.row == 48 and GqaDims(2, 1, 8, 8, 4, 1.0, 1e-5, norm=False).turned
    t = [torch.tensor(x) for x in ([1.0, 2.0], [0.5, 0.25], [0.1, 0.2], [1.0, -1.0])]
    assert math.isclose(differential_blend(*t, 0.25), math.e - math.exp(0.1 * 1.0 - 0.2) + 0.25, rel_tol=1e-6) and GqaWeights.pack(D, None, None, "cpu", blend=0.5).blend == 0.5
    base = dict(uk=torch.ones(20, 20), uv=torch.ones(14, 20), out=torch.ones(6, 14), device="cpu", dtype=torch.float32)
    for gate, rot, rows in ((GATE_HEAD, 0, 2), (GATE_ELEMENT, 4, 14)):
        L = LatentDims(2, 10, rot, 7, 20, 0.3, 1e-5, gate=gate)
        heads = 2 * (16 + (8 if rot else 0))
        assert (L.q_cols, L.gate_col, L.gate_cols, L.proj_cols) == (heads, heads + 24 + (8 if rot else 0), 16 if rot else 2, heads + 24 + (8 if rot else 0) + (16 if rot else 8))
        g = torch.arange(1.0, rows + 1).reshape(-1, 1) @ torch.ones(1, 6)
        w = LatentWeights.pack(L, torch.ones(2 * (10 + rot), 6), torch.ones(20 + rot, 6), torch.ones(20), gate=g, **base)
        assert w.proj[L.gate_col:, 0].tolist() == ([*range(1, 8), 0, *range(8, 15), 0] if rot else [1, 2, 0, 0, 0, 0, 0, 0])
        with pytest.raises(InvalidArgument):
            LatentWeights.pack(L, torch.ones(2 * (10 + rot), 6), torch.ones(20 + rot, 6), torch.ones(20), **base)
    with pytest.raises(InvalidArgument):
        LatentWeights.pack(LatentDims(2, 10, 0, 7, 20, 0.3, 1e-5), torch.ones(20, 6), torch.ones(20, 6), torch.ones(20), gate=torch.ones(2, 6), **base)
    d = DensePolyWeights.pack(torch.ones(9, 5), 2 * torch.ones(5, 9), torch.arange(4.0), 0.5, "cpu", torch.float32)
    assert d.up.stride() == (32, 1) and d.down.shape == (5, 9) and d.down.stride(0) == 32 and d.coef.tolist() == [0, 1, 2, 3] and (d.ff, d.eps) == (9, 0.5)
    r = RouteRule(torch.zeros(8), softmax=True)
    assert MoeWeights(torch.zeros(4, 8), None, None, 8, 2, form="silu", rule=r).rule_args == (2, r.correction, 0, 0, 1.0)


def test_size_limits_of_the_kernels():
    L = _lib.kernels()
    # dim, vdim -> whether one CTA takes both maps, sub-tiles
    for d, dv, joins, sub in ((16, 16, 1, 1), (64, 128, 1, 1), (65, 128, 1, 1), (128, 128, 1, 1), (129, 64, 0, 2), (129, 128, 0, 2), (64, 129, 0, 1), (64, 256, 0, 1), (64, 257, 0, 0), (300, 60, 0, 1), (512, 200, 0, 0)):
        assert L.ft_gqa_flash_joins_maps(d, dv) == joins, (d, dv)
        assert L.ft_gqa_flash_subtiles(4, 2, d, dv, 2) == sub, (d, dv)
    assert L.ft_gqa_flash_subtiles(300, 2, 64, 64, 2) == 0 and L.ft_gqa_flash_subtiles(4, 2, 64, 64, 3) == 0
    D = GqaDims(6, 2, 40, 72, 0, 1.0, 1e-5, norm=False, maps=2)
    assert D.flash_tile() == 128 // 3 and D.decode_supported()
    assert GqaDims(2, 2, 128, 256, 0, 1.0, 1e-5, norm=False, maps=2).decode_supported() and not GqaDims(2, 2, 128, 528, 0, 1.0, 1e-5, norm=False, maps=2).decode_supported()


def test_the_shift_finds_the_rows_and_slot_of_every_sequence():
    s = StateSlots(4, [8, 8])
    c = PagedRowCache(PagePool(100, 16), [16, 0], states=s)
    lens, starts = [40, 1, 30], [0, 9, 17]
    for k, (n, st) in enumerate(zip(lens, starts)):
        c.add_sequence(k)
        c.reserve(k, n + st)
        c.lengths[k] = st
    b = RowBatch([StepEntry(k, [0] * n) for k, n in enumerate(lens)], c, "cpu", 100)
    p = b.memory_plan(0)
    assert p.spans.tolist() == [[0, 40, s.slot[0], 1], [40, 1, s.slot[1], 0], [41, 30, s.slot[2], 0]] and p.spans.data_ptr() % 16 == 0
    assert b.seq_of.tolist() == [0] * 40 + [1] + [2] * 30
