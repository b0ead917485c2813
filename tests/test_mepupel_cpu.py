"""Host side of the Mepupel decoder: configuration, registry, weight packing, rotation frequencies, batch tables, size limits, and the plain reference against closed forms."""
import json
import math

import numpy as np
import pytest
import torch

import mepupel_oracle as O
from ferrotorch_b200 import _build, _lib
from ferrotorch_b200.errors import InvalidArgument, ShapeMismatch
from ferrotorch_b200.models import (AttentionConfig, DenseConfig, ExpertConfig, GinisunConfig, LatentConfig, Mamba2Config, MepupelConfig, MepupelLayer, MepupelModel, MoeConfig, PufevikConfig,
                                    RandomMepupelWeights, RowBatch, StepEntry, architectures, load_model_config, registry)
from ferrotorch_b200.nn import PagedRowCache, PagePool, StateSlots
from ferrotorch_b200.ops import DenseGatedWeights, GqaDims, GqaWeights, LatentDims, LatentWeights, MoeWeights, RouteRule, SsmDims, SsmWeights
from ferrotorch_b200.ops.gqa_attention import NORM_HEAD, NORM_NONE, NORM_WHOLE
from ferrotorch_b200.ops.latent_attention import rotary_pair_tables

YARN = dict(factor=4.0, original=64, fast=8.0, slow=1.0)


def test_configuration_reads_every_size_of_every_layer():
    cfg, W = O.random_model(3, kinds="malla", scaling=YARN, overrides={0: dict(mlp="dense", ff=11, conv=2, norm_groups=8), 1: dict(mlp=None, window=77, keep_first=5), 3: dict(kv_from=2, lat_heads=7, q_rank=3),
                                                                       4: dict(rot=0, window=0, scale=0.7, group_count=0, shared=0, router_scale=1.0)})
    c = MepupelConfig.from_dict(cfg)
    assert {k: tuple(v.shape) for k, v in W.items()} == c.tensor_shapes()
    assert c.layers[0] == MepupelLayer(Mamba2Config(4, 16, 24, 2, 8, 2), DenseConfig(11)) and "l0.mlp.up.b" in W
    assert c.layers[1] == MepupelLayer(AttentionConfig(4, 2, 16, 24, 0.25, 8, 10000.0, 77, False, 5, {k: float(v) for k, v in YARN.items()}), None) and "l1.norm2" not in W
    moe = MoeConfig(8, 3, ExpertConfig(40), ExpertConfig(24), 4, 2, 1.7)
    assert c.layers[2] == MepupelLayer(LatentConfig(3, 16, 20, 24, 32, 0.25), moe) and c.layers[3] == MepupelLayer(LatentConfig(7, 16, 20, 3, 32, 0.25, 2), moe)
    assert "l2.mix.dkv" in W and "l3.mix.dkv" not in W and c.latent_source(3) == 2 and c.latent_source(2) == 2
    assert c.layers[4].mixer == AttentionConfig(4, 2, 16, 24, 0.7) and c.layers[4].mlp == MoeConfig(8, 3, ExpertConfig(40)) and "l4.mlp.shared.up" not in W
    assert c.residual_mult == 0.4 and c.vocab_size == 90 and c.layers[0].mixer.channels == 64 + 2 * 2 * 24
    assert MepupelConfig.from_dict(json.loads(json.dumps(c.to_dict()))) == c
    r = RandomMepupelWeights(c, device="cpu")
    assert all(tuple(r[k].shape) == s and r[k].dtype == torch.bfloat16 for k, s in c.tensor_shapes().items()) and "l0.mix.D" in r


def _set(i, part, **kw):
    return lambda c: c["layers"][i][part].update(**kw)


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="other"), _set(0, "mixer", groups=3), _set(0, "mixer", norm_groups=5), _set(0, "mixer", conv=0), _set(1, "mixer", heads=3),
                                    _set(1, "mixer", rot=dict(base=1e4, dims=7)), _set(1, "mixer", mask=dict(size=4, keep_first=-1)), _set(1, "mixer", v_mix=True), _set(1, "mixer", scale=0.0),
                                    _set(1, "mixer", rot=dict(base=1e4, dims=8, scaling=dict(factor=0.0, original=64, fast=8, slow=1))), _set(2, "mixer", q_rank=0), _set(3, "mixer", kv_from=1),
                                    _set(3, "mixer", kv_from=3), _set(3, "mixer", kv_rank=33), _set(2, "mixer", kv_from=3), _set(0, "mlp", kind="other"),
                                    lambda c: c["layers"][0]["mlp"]["router"].update(top=9), lambda c: c["layers"][0]["mlp"]["router"].update(groups=dict(count=3, keep=1)),
                                    lambda c: c["layers"][0]["mlp"]["router"].update(groups=dict(count=4, keep=1)), lambda c: c["layers"][0]["mlp"]["router"].update(groups=dict(count=4, keep=5)),
                                    lambda c: c["layers"][0]["mlp"]["expert"].update(limit=2.0), lambda c: c.update(layers=[]), lambda c: c.update(vocab=0)])
def test_configuration_refuses_what_it_cannot_run(change):
    cfg, _ = O.random_model(1, kinds="mall", overrides={3: dict(kv_from=2)})
    MepupelConfig.from_dict(cfg)
    change(cfg)
    with pytest.raises(InvalidArgument):
        MepupelConfig.from_dict(cfg)


def test_a_latent_is_borrowed_from_its_owner_only():
    cfg, _ = O.random_model(1, kinds="lll", overrides={1: dict(kv_from=0), 2: dict(kv_from=1)})
    with pytest.raises(InvalidArgument):
        MepupelConfig.from_dict(cfg)


def test_other_designs_refuse_the_constants_they_do_not_have():
    att = dict(heads=2, kv_heads=1, dim=8, vdim=8, scale=1.0, rot=dict(dims=4, base=10.0))
    for extra in (dict(mask=dict(size=4, keep_first=2)), dict(rot=dict(dims=4, base=10.0, scaling=YARN))):
        with pytest.raises(InvalidArgument):
            PufevikConfig.from_dict(dict(vocab=4, width=8, norm=dict(eps=1e-5), embedding=dict(scale=1.0), layers=[dict(
                type="parallel", mixer=dict(left=dict(att, **extra), right=dict(heads=1, dim=8, vdim=8, gate_cap=1.0), left_scale=1.0, right_scale=1.0), mlp=None)]))
    g = GinisunConfig.uniform(1, 8, 8, 1, 8, 4, 8, 8, 4, 2, 8).to_dict()
    GinisunConfig.from_dict(g)
    for extra in (dict(groups=dict(count=2, keep=1)), dict(scale=2.0)):
        with pytest.raises(InvalidArgument):
            h = json.loads(json.dumps(g))
            h["layers"][0]["mlp"]["router"].update(extra)
            GinisunConfig.from_dict(h)


def test_registry_weights_and_device(tmp_path):
    cfg, W = O.random_model(1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    arch, c = load_model_config(tmp_path)
    assert arch.name == "Mepupel" and isinstance(c, MepupelConfig) and "Mepupel" in architectures()
    with pytest.raises(InvalidArgument):
        MepupelModel(c, {k: torch.tensor(v) for k, v in W.items()}, device="cpu")
    with pytest.raises(ShapeMismatch):
        get = registry.checked_weights("Mepupel", c.tensor_shapes(), {**{k: torch.tensor(v) for k, v in W.items()}, "l0.mix.conv": torch.zeros(3, 3)}, "cpu")
        get("l0.mix.conv")


def test_a_partial_kernel_library_is_complete():
    """The sources that the architecture names link without the rest."""
    import ctypes
    lib = _build.build_kernels_part("mepupel_test", registry._ARCHITECTURES["mepupel"].kernels)
    try:
        h = ctypes.CDLL(str(lib))          # unresolved symbols would show here
        assert h.ft_abi_version() == 1 and all(hasattr(h, n) for n in ("ft_ssm_walk", "ft_gqa_flash", "ft_latent_flash", "ft_moe_topk", "ft_parallel_update")) and not hasattr(h, "ft_mm_walk")
    finally:
        lib.unlink()


@pytest.mark.parametrize("dims,base,scaling", [(24, 5e5, dict(factor=10.0, original=3000, fast=20.0, slow=1.5)), (16, 700.0, YARN), (6, 50.0, dict(factor=1.5, original=30, fast=2.0, slow=0.1)),
                                               (8, 1e4, dict(factor=0.5, original=7, fast=1.0, slow=1.0)), (4, 3.0, dict(factor=16.0, original=1e6, fast=1.0, slow=1e-9)), (10, 100.0, None)])
def test_rotation_tables_follow_the_scaling(dims, base, scaling):
    """Also where the ramp has no width, or starts past the last pair."""
    a = AttentionConfig(1, 1, dims, 8, 1.0, dims, base, scaling=scaling)
    cos, sin = rotary_pair_tables(200, dims, base, "cpu", a.rope_scaling)
    f, k = O.frequencies(dims, base, scaling)
    ang = np.arange(200)[:, None] * f[None]
    assert np.abs(cos.double().numpy() - k * np.cos(ang)).max() < 1e-6 and np.abs(sin.double().numpy() - k * np.sin(ang)).max() < 1e-6


def test_the_reference_agrees_with_closed_forms():
    rng = np.random.default_rng(0)
    # state space: a stretch at once
    x, B, C, d = rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 1, 4)), rng.standard_normal((9, 1, 4)), rng.random((9, 2))
    A, D = rng.standard_normal(2), rng.standard_normal(2)
    y, S = O.state_space(x, B, C, d, A, D)
    for h in range(2):
        F = np.cumsum(-np.exp(A[h]) * d[:, h])
        w = np.tril((C[:, 0] @ B[:, 0].T) * np.exp(np.minimum(F[:, None] - F[None], 0.0)) * d[None, :, h])
        assert np.allclose(y[:, h], w @ x[:, h] + D[h] * x[:, h])
        assert np.allclose(S[h], (np.exp(F[-1] - F) * d[:, h] * B[:, 0].T) @ x[:, h])
    # convolution as numpy's
    u, w, b = rng.standard_normal((7, 2)), rng.standard_normal((2, 3)), rng.standard_normal(2)
    got = O.causal_convolution(u, w, b)
    for c in range(2):
        assert np.allclose(got[:, c], np.convolve(u[:, c], w[c, ::-1])[:7] + b[c])
    # masks by hand
    see = O.visible(7, 3, 2)
    assert [[j for j in range(7) if see[i, j]] for i in (0, 2, 3, 6)] == [[0], [0, 1, 2], [0, 1, 2, 3], [0, 1, 4, 5, 6]]
    # rotation keeps lengths (times the factor) and depends on distances only
    q, k = rng.standard_normal((2, 1, 1, 6))
    a, b = (O.rotate_halves(q, [p], 4, 30.0, YARN) * O.rotate_halves(k, [p - 3], 4, 30.0, YARN) for p in (3, 40))
    assert np.isclose(a[..., :4].sum(), b[..., :4].sum()) and np.allclose(O.rotate_halves(q, [9], 4, 30.0)[..., 4:], q[..., 4:])
    # the gated norm's parts
    g = O.gated_group_norm(np.ones((1, 6)) * [1, 1, 1, 5, 5, 5], np.full((1, 6), 50.0), np.ones(6), 2, 0.0)
    assert np.allclose(g, 1.0)


def test_packed_weights_keep_every_row_where_the_kernels_look():
    D = SsmDims(3, 5, 7, 1, 2, 5, 1e-5)
    assert (D.v16, D.n16, D.h8, D.out_cols, D.channels, D.main, D.state_size) == (16, 16, 8, 48, 80, 128, 3 * 256 + 80)
    ch = 15 + 14
    w = torch.arange(1.0, 15 + ch + 3 + 1).reshape(-1, 1) @ torch.ones(1, 4)
    p = SsmWeights.pack_projection(D, w, "cpu", torch.float32)[:, 0]
    assert p.shape == (136,) and p[:5].tolist() == [1, 2, 3, 4, 5] and p[16:21].tolist() == [6, 7, 8, 9, 10] and float(p[5:16].sum()) == 0
    assert p[48:53].tolist() == [16, 17, 18, 19, 20] and p[96:103].tolist() == list(range(31, 38)) and p[112:119].tolist() == list(range(38, 45)) and p[128:131].tolist() == [45, 46, 47]
    v = SsmWeights.pack(D, torch.arange(2.0 * ch).reshape(ch, 2), torch.arange(1.0 * ch), torch.ones(3), torch.zeros(3), torch.ones(3), torch.ones(15), "cpu")
    assert v.conv.shape == (2, 80) and v.conv[:, 17].tolist() == [12, 13] and v.conv_bias[16] == 5 and v.rate.tolist() == [-1] * 3 + [0] * 5 and float(v.norm.sum()) == 15
    L = LatentDims(2, 10, 0, 7, 20, 0.3, 1e-5, q_rank=13)
    assert (L.row, L.q_cols, L.proj_cols) == (32, 16, 40) and LatentDims(2, 10, 0, 7, 20, 0.3, 1e-5, 13, False).proj_cols == 16
    t = dict(uk=torch.ones(20, 20), uv=torch.ones(14, 20), out=torch.ones(6, 14))
    lw = LatentWeights.pack(L, torch.ones(20, 13), 2 * torch.ones(20, 6), torch.ones(20), **t, device="cpu", dtype=torch.float32, dq=3 * torch.ones(13, 6), q_norm=torch.ones(13))
    assert lw.proj[:, 0].tolist() == [3] * 13 + [0] * 3 + [2] * 20 + [0] * 4 and lw.uq.shape == (32, 13) and lw.uq[:, 0].tolist() == ([1] * 10 + [0] * 6) * 2 and lw.q_norm.shape == (16,)
    for bad in (dict(dq=None, q_norm=None), dict(dkv=None, norm=None)):
        kw = dict(dq=torch.ones(13, 6), q_norm=torch.ones(13), dkv=torch.ones(20, 6), norm=torch.ones(20))
        kw.update(bad)
        with pytest.raises(InvalidArgument):
            LatentWeights.pack(L, torch.ones(20, 13), **t, device="cpu", dtype=torch.float32, **kw)
    g = GqaWeights.pack(GqaDims(2, 1, 8, 8, 4, 1.0, 1e-5, norm=False), None, None, "cpu")
    assert g.q_norm is None and [GqaDims(2, 1, 8, 8, 4, 1.0, 1e-5, whole_norm=a, norm=b).norm_kind for a, b in ((False, True), (True, True), (True, False))] == [NORM_HEAD, NORM_WHOLE, NORM_NONE]
    d = DenseGatedWeights.pack(torch.ones(9, 5), torch.ones(9, 5), torch.ones(5, 9), "cpu", torch.float32, "silu", torch.arange(1.0, 10), 10 * torch.arange(1.0, 10), torch.ones(5))
    assert d.gu_bias.tolist() == [*range(1, 9), *range(10, 90, 10), 9] + [0] * 7 + [90] + [0] * 7 and d.down_bias.tolist() == [1] * 5 + [0] * 3
    m = MoeWeights(torch.zeros(4, 8), None, None, 8, 2)
    assert m.rule_args == (0, None, 0, 0, 1.0) and m.kind == 0
    r = RouteRule(torch.zeros(8), 2, 1, 1.5)
    assert MoeWeights(torch.zeros(4, 8), None, None, 8, 2, form="silu", rule=r).rule_args == (1, r.correction, 2, 1, 1.5)


def test_size_limits_of_the_kernels():
    L = _lib.kernels()
    for d, dv in ((16, 16), (64, 64), (65, 64), (128, 128), (128, 64), (192, 128), (64, 200), (300, 16)):
        assert LatentDims(2, d, 0, dv, 64, 1.0, 1e-5, 16).flash_tile() == L.ft_latent_flash_tile(d, 0, dv), (d, dv)
    assert SsmDims(1, 999, 256, 1, 4, 1, 1e-5).walk_supported() and not SsmDims(1, 16, 257, 1, 4, 1, 1e-5).walk_supported()
    assert SsmDims(1, 16, 4096, 1, 4, 1, 1e-5).decode_supported() and not SsmDims(1, 16, 4097, 1, 4, 1, 1e-5).decode_supported()
    for bad in (SsmDims(4, 16, 16, 3, 4, 1, 1e-5), SsmDims(4, 16, 16, 2, 4, 7, 1e-5), SsmDims(2000, 16, 16, 1, 4, 1, 1e-5), SsmDims(4, 16, 0, 2, 4, 1, 1e-5)):
        with pytest.raises(InvalidArgument):
            bad.validate()


@pytest.mark.parametrize("ctas", [0, 1, 32])
def test_plans_name_the_rows_and_slot_of_every_sequence(ctas):
    s = StateSlots(4, [4])
    c = PagedRowCache(PagePool(600, 16), [0], states=s)
    lens, starts = [1000, 3, 300], [0, 9, 17]
    for k, (n, st) in enumerate(zip(lens, starts)):
        c.add_sequence(k)
        c.reserve(k, n + st)
        c.lengths[k] = st
    p = RowBatch([StepEntry(k, [0] * n) for k, n in enumerate(lens)], c, "cpu", 600).memory_plan(ctas)
    assert p.spans.tolist() == [[0, 1000, s.slot[0], 1], [1000, 3, s.slot[1], 0], [1003, 300, s.slot[2], 0]]
    assert p.spans.data_ptr() % 16 == 0 and p.chains.data_ptr() % 16 == 0
    c.fork(0, "fork")                       # layers without rows: a page is copied without them
    c.reserve("fork", 1001)
    assert c.rows[0].shape[-1] == 0


def test_scaling_constants_of_the_configuration():
    a = AttentionConfig.from_dict(dict(heads=2, kv_heads=1, dim=8, vdim=8, scale=0.5, rot=dict(dims=4, base=9.0, scaling=YARN)))
    assert a.rope_scaling["attention_factor"] == 0.1 * math.log(4.0) + 1.0 and AttentionConfig(2, 1, 8, 8, 0.5).rope_scaling is None
