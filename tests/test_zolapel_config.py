"""Zolapel on the CPU: the configuration reader, the manifest, the order of runs and their caches, and the plain implementation's own pieces."""
import copy

import numpy as np
import pytest
import torch

import plain_zolapel as PZ
import zolapel_models as ZM
from vitna_anchor_b200.config import ConfigError, resolve
from vitna_anchor_b200.config.zolapel import ZolapelConfig
from vitna_anchor_b200.models.zolapel import is_norm_weight, zolapel_manifest
from vitna_anchor_b200.parts.rotary import banded_frequencies
from vitna_anchor_b200.weights.random_init import random_weights


@pytest.mark.parametrize("name", sorted(ZM.CONFIGS))
def test_config_reads_back_and_names_every_tensor(name):
    cj = ZM.CONFIGS[name]
    arch = resolve(cj)
    assert arch.name == "Zolapel"
    cfg = arch.parse_config(cj)
    assert ZolapelConfig.from_dict(cfg.to_dict()) == cfg
    made = ZM.make_tensors(cj, 0)
    specs = {w.name: w for w in zolapel_manifest(cfg)}
    assert set(specs) == set(made)
    for n, t in made.items():
        assert specs[n].fits(t.shape), n


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="parallel"), "type"),
    (lambda c: c["layers"][0].update(extra=1), "extra"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=3.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(scale=-1.0), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(style="halves"), "style"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("low"), "low"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(low=5.0), "scaling"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), "scaling"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(first=2), "first"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][1]["mlp"].update(shared={}), "shared"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(scale=2.0), "scale"),
    (lambda c: c["token_side"].update(norm=1), "norm"),
    (lambda c: c["token_side"].pop("dim"), "dim"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(residual_mult="half"), "residual_mult"),
])
def test_what_the_engine_does_not_have_is_refused_by_name(change, word):
    cj = copy.deepcopy(ZM.CONFIGS["all"])
    change(cj)
    with pytest.raises(ConfigError, match=word):
        ZolapelConfig.from_dict(cj)


def test_what_may_be_left_out():
    cj = copy.deepcopy(ZM.CONFIGS["all"])
    del cj["loop"], cj["token_side"], cj["residual_mult"]
    for key in ("kv_heads", "vdim", "rot", "mask"):
        del cj["layers"][0]["mixer"][key]
    cfg = ZolapelConfig.from_dict(cj)
    m = cfg.layers[0].mixer
    assert (m.kv_heads, m.rot, m.window, cfg.residual_mult, cfg.side_dim) == (4, None, 0, 1.0, 0)
    assert cfg.layers[1].mixer.rot.scaling is None and cfg.layers[2].mlp is None
    names = {w.name for w in zolapel_manifest(cfg)}
    assert not {"loop.step", "side.embed", "l0.side.gate", "l2.norm2", "l2.ls2"} & names and "l2.ls1" in names


def test_every_run_has_pages_of_its_own_and_every_pass_its_vector():
    arch = resolve(ZM.CFG_ALL)
    cfg = arch.parse_config(ZM.CFG_ALL)
    assert cfg.runs() == PZ.runs(ZM.CFG_ALL) == [(0, -1), (1, 0), (2, -1), (1, 1), (2, -1), (1, 2), (2, -1), (3, -1)]
    t = ZM.make_tensors(ZM.CFG_ALL, 1)
    model = arch.build(cfg, {k: torch.from_numpy(v) for k, v in t.items()}, torch.float32, "cpu")
    assert [r.block for r in model.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert sorted(r.cache for r in model.schedule) == list(range(8)) and all(r.state < 0 for r in model.schedule)
    begins = [r.before for r in model.schedule if r.before is not None]
    assert [r.before is not None for r in model.schedule] == [False, True, False, True, False, True, False, False]
    assert [b.table is not None for b in begins] == [False, True, True]
    for k, b in enumerate(begins):
        assert np.array_equal(b.step.numpy(), t["loop.step"][k])
    assert model.capture_safe and model.lm_head.weight.data_ptr() == model.embedding.table.data_ptr()
    per = [b.weight_bytes() for b in model.blocks]
    assert model.step_weight_bytes() == (per[0] + 3 * (per[1] + per[2]) + per[3] + 3 * 4 * 64 + model.final_norm.weight_bytes() + model.lm_head.weight_bytes())


def test_the_parts_hold_what_the_checkpoint_has():
    arch = resolve(ZM.CFG_ODD)
    t = ZM.make_tensors(ZM.CFG_ODD, 2)
    model = arch.build(arch.parse_config(ZM.CFG_ODD), {k: torch.from_numpy(v) for k, v in t.items()}, torch.float32, "cpu")
    b = model.blocks[0]
    rows = np.concatenate([t["l0.mix.q"], t["l0.mix.k"], t["l0.mix.g"]])
    assert b.mixer.cols == 40 and b.mixer.w_in.shape[0] % 4 == 0
    assert np.array_equal(b.mixer.w_in.numpy()[:43], rows) and not b.mixer.w_in.numpy()[43:].any()
    assert np.allclose(b.mixer_scale.numpy(), 1.3 * t["l0.ls1"], rtol=1e-6) and np.allclose(b.ffn_scale.numpy(), 1.3 * t["l0.ls2"], rtol=1e-6)
    assert np.array_equal(b.ffn.w_gate_up[2].numpy(), t["l0.mlp.e2.up"]) and np.array_equal(b.ffn.w_down[1].numpy(), t["l0.mlp.e1.down"])
    assert b.side is None


def test_parts_that_do_not_fit_are_refused():
    from vitna_anchor_b200.parts.block import ScaledResidualBlock, TokenSide
    from vitna_anchor_b200.parts.feed_forward import RoutedExperts, ScoredRouter
    from vitna_anchor_b200.parts.loop import PassOffset
    from vitna_anchor_b200.parts.norms import LayerNorm
    from vitna_anchor_b200.parts.rotary_attention import RotaryAttention
    z = lambda *s: torch.zeros(*s)
    with pytest.raises(ValueError, match="keys' size"):
        RotaryAttention(8, 1, 1, 4, 6, 1.0, z(8, 8), z(8, 6), v_from_k=True)
    with pytest.raises(ValueError, match="head counts"):
        RotaryAttention(8, 2, 1, 4, 4, 1.0, z(16, 8), z(8, 8), gate=True)
    with pytest.raises(ValueError, match="come together"):
        RotaryAttention(8, 1, 1, 4, 4, 1.0, z(12, 8), z(8, 4), q_norm=z(4), eps=1e-5)
    with pytest.raises(ValueError, match="inputs"):
        RoutedExperts(8, 4, 2, 1, z(2, 8), None, z(2, 4, 8), z(2, 8, 4), activation="gelu", gated=False, weigh_input=True, scored=ScoredRouter(sigmoid=True))
    with pytest.raises(ValueError, match="width"):
        PassOffset(8, z(4))
    with pytest.raises(ValueError, match="per-layer"):
        TokenSide(8, z(4, 8), z(8, 4), z(10, 8), 6, z(8), 1e-5)
    ln = lambda eps: LayerNorm(8, eps, z(8), z(8))
    mixer = RotaryAttention(8, 1, 1, 4, 4, 1.0, z(12, 8), z(8, 4))
    with pytest.raises(ValueError, match="come together"):
        ScaledResidualBlock(ln(1e-5), mixer, z(8), ffn_norm=ln(1e-5))
    with pytest.raises(ValueError, match="one eps"):
        ScaledResidualBlock(ln(1e-5), mixer, z(8), side=TokenSide(8, z(4, 8), z(8, 4), z(10, 8), 4, z(8), 1e-6))


def test_random_weights_of_the_design():
    cfg = ZolapelConfig.from_dict(ZM.CFG_ALL)
    w = random_weights(zolapel_manifest(cfg), 3, is_norm=is_norm_weight)
    for name in ("l0.norm1", "l1.norm2", "l0.mix.q.norm", "l0.mix.k.norm", "l3.side.norm", "final.norm", "l0.ls1", "l3.ls2"):
        assert float(w[name].float().mean()) == 1.0, name
    for name in ("l0.norm1.b", "final.norm.b", "loop.step", "l0.mix.g", "l1.mlp.router"):
        assert abs(float(w[name].float().mean())) < 0.1, name


def test_frequencies_are_kept_divided_and_blended():
    for base, dims, sc in ((10000.0, 32, dict(factor=8.0, low=1.0, high=4.0, original=64)), (500.0, 10, dict(factor=3.0, low=2.0, high=2.0, original=100)),
                           (50.0, 6, None), (7.0, 2, dict(factor=2.0, low=0.5, high=32.0, original=9))):
        got = banded_frequencies(base, dims, None if sc is None else tuple(sc[k] for k in ("factor", "low", "high", "original")))
        assert got.dtype == np.float32 and np.allclose(got, PZ.frequencies(base, dims, sc), rtol=2e-7)
    f = base_f = np.array([10000.0 ** (-i / 16.0) for i in range(16)])
    got = PZ.frequencies(10000.0, 32, dict(factor=8.0, low=1.0, high=4.0, original=64))
    length = 2 * np.pi / f
    assert np.array_equal(got[length < 16], base_f[length < 16]) and np.allclose(got[length > 64], base_f[length > 64] / 8)
    between = (length > 16) & (length < 64)
    assert between.any() and (got[between] < base_f[between]).all() and (got[between] > base_f[between] / 8).all()
    # half-way between the two edges in original / wavelength: the mean of the two frequencies
    one = PZ.frequencies(2 * np.pi / 25.6, 0, None)
    assert len(one) == 0
    mid = PZ.frequencies((64 / 2.5 / (2 * np.pi)) ** 2.0, 4, dict(factor=8.0, low=1.0, high=4.0, original=64))[1]
    assert np.isclose(mid, 0.5 * (2 * np.pi * 2.5 / 64) * (1 + 1 / 8))


def test_the_plain_pieces():
    x = np.random.default_rng(0).standard_normal((3, 5, 12))
    f = PZ.frequencies(50.0, 8)
    y = PZ.turn_neighbours(x, np.arange(5), f)
    assert np.array_equal(y[..., 8:], x[..., 8:]) and np.array_equal(y[:, 0], x[:, 0])
    assert np.allclose(y[:, 2, 2], x[:, 2, 2] * np.cos(2 * f[1]) - x[:, 2, 3] * np.sin(2 * f[1]))
    assert np.allclose(y[:, 2, 3], x[:, 2, 3] * np.cos(2 * f[1]) + x[:, 2, 2] * np.sin(2 * f[1]))
    # a weight on an expert's input is its square on the output: relu squared is homogeneous of degree 2
    cfg = ZM.config(30, 16, [ZM.layer(ZM.att(1, 1, 4, 0.5), ZM.moe(8, 3, 1))])
    w = {k: v.astype(np.float64) for k, v in ZM.make_tensors(cfg, 1).items()}
    h = np.random.default_rng(2).standard_normal((4, 16))
    assert np.allclose(PZ.expert(w, "l0.mlp.e1.", 0.3 * h), 0.09 * PZ.expert(w, "l0.mlp.e1.", h), rtol=1e-12)
    got = PZ.experts_ff(w, "l0.mlp.", cfg["layers"][0]["mlp"], h)
    s = 1 / (1 + np.exp(-h @ w["l0.mlp.router"].T))
    for t in range(4):
        e = int(np.argmax(s[t]))
        assert np.allclose(got[t], PZ.expert(w, f"l0.mlp.e{e}.", s[t, e] * h[t]))
    # no key but the query's own: the head's output is its own projected key, gated
    m = ZM.att(2, 1, 4, 0.5, (10.0, 4), 1)
    v = h @ w["l0.mix.k"].T
    w2 = dict(w, **{"l0.mix.q": np.random.default_rng(3).standard_normal((8, 16)), "l0.mix.g": np.random.default_rng(4).standard_normal((2, 16)),
                    "l0.mix.o": np.eye(8)})
    g = 1 / (1 + np.exp(-h @ w2["l0.mix.g"].T))
    assert np.allclose(PZ.attention(w2, "l0.mix.", m, h, 1e-5), np.concatenate([g[:, :1] * v, g[:, 1:] * v], axis=1))
