"""Lirutar on the CPU: the configuration reader, the manifest, the order of runs and their caches, and the plain implementation's own pieces."""
import copy

import numpy as np
import pytest
import torch

import lirutar_models as LM
import plain_lirutar as PL
from vitna_anchor_b200.config import ConfigError, resolve
from vitna_anchor_b200.config.lirutar import LirutarConfig
from vitna_anchor_b200.models.lirutar import _frequencies, is_norm_weight, lirutar_manifest
from vitna_anchor_b200.weights.random_init import random_weights


@pytest.mark.parametrize("name", sorted(LM.CONFIGS))
def test_config_reads_back_and_names_every_tensor(name):
    cj = LM.CONFIGS[name]
    arch = resolve(cj)
    assert arch.name == "Lirutar"
    cfg = arch.parse_config(cj)
    assert LirutarConfig.from_dict(cfg.to_dict()) == cfg
    made = LM.make_tensors(cj, 0)
    specs = {w.name: w for w in lirutar_manifest(cfg)}
    assert set(specs) == set(made)
    for n, t in made.items():
        assert specs[n].fits(t.shape), n


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(middle={}), "middle"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=3.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(scale=0.0), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=5), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(factor=2.0), "factor"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(groups=3), "groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(dim=5), "dim"),
    (lambda c: c["layers"][0]["mlp"].update(limit=1.0), "limit"),
    (lambda c: c["layers"][1]["mlp"].update(kind="experts"), "kind"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3), "count"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=5), "keep"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_what_the_engine_does_not_have_is_refused_by_name(change, word):
    cj = copy.deepcopy(LM.CONFIGS["all"])
    change(cj)
    with pytest.raises(ConfigError, match=word):
        LirutarConfig.from_dict(cj)


def test_what_may_be_left_out():
    cj = copy.deepcopy(LM.CONFIGS["all"])
    del cj["loop"], cj["layers"][0]["mixer"]["left"]["kv_heads"], cj["layers"][0]["mixer"]["left"]["vdim"], cj["layers"][0]["mixer"]["left_scale"]
    del cj["layers"][3]["mlp"]["router"]["groups"], cj["layers"][3]["mlp"]["router"]["identity"], cj["layers"][3]["mlp"]["router"]["scale"]
    cfg = LirutarConfig.from_dict(cj)
    left = cfg.layers[0].mixer.left
    assert left.kv_heads == 4 and left.vdim == 16 and cfg.layers[0].mixer.left_scale == 1.0
    r = cfg.layers[3].mlp
    assert (r.count, r.keep, r.identity, r.scale, r.shared) == (1, 1, 0, 1.0, None)
    assert cfg.layers[3].mixer.left.window == 0 and cfg.layers[2].mixer.left.rot is None and cfg.layers[2].mlp is None
    assert not any(w.name == "loop.in" for w in lirutar_manifest(cfg))


def test_every_run_has_pages_and_a_state_of_its_own():
    arch = resolve(LM.CFG_ALL)
    cfg = arch.parse_config(LM.CFG_ALL)
    assert cfg.runs() == PL.runs(LM.CFG_ALL) == [(0, False)] + [(1, True), (2, False)] * 3 + [(3, False)]
    made = {k: torch.from_numpy(v) for k, v in LM.make_tensors(LM.CFG_ALL, 1).items()}
    model = arch.build(cfg, made, torch.float32, "cpu")
    assert [r.block for r in model.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    places = [r.cache for r in model.schedule] + [r.state for r in model.schedule]
    assert sorted(places) == list(range(16))
    assert [r.before is not None for r in model.schedule] == [False, True, False, True, False, True, False, False]
    assert len(model.entries) == 1 and model.capture_safe
    # what a step reads: a block as often as it runs, and the matrix in front of a pass as often as there are passes
    per = [b.weight_bytes() for b in model.blocks]
    assert model.step_weight_bytes() == (per[0] + 3 * per[1] + 3 * per[2] + per[3] + 3 * model.entries[0].weight_bytes()
                                         + model.final_norm.weight_bytes() + model.lm_head.weight_bytes())


def test_the_pair_stacks_both_products():
    """The input matrices by rows, the output matrices side by side, as the checkpoint has them (the scales are not folded in)."""
    arch = resolve(LM.CFG_ODD)
    t = LM.make_tensors(LM.CFG_ODD, 2)
    model = arch.build(arch.parse_config(LM.CFG_ODD), {k: torch.from_numpy(v) for k, v in t.items()}, torch.float32, "cpu")
    mx = model.blocks[1].mixer
    rows = np.concatenate([t["l1.mix.left.q"], t["l1.mix.left.k"], t["l1.mix.left.v"], t["l1.mix.right.in"]])
    assert np.array_equal(mx.w_in.numpy(), rows)
    assert np.array_equal(mx.w_out.numpy(), np.concatenate([t["l1.mix.left.o"], t["l1.mix.right.o"]], axis=1))
    assert (mx.left_scale, mx.right_scale) == (1.4, 0.3)


def test_mixers_that_cannot_stand_side_by_side_are_refused():
    from vitna_anchor_b200.parts.parallel import ParallelMixer
    from vitna_anchor_b200.parts.rotary_attention import RotaryAttention
    z = lambda *s: torch.zeros(*s)
    a = lambda w: RotaryAttention(w, 1, 1, 4, 4, 1.0, z(12, w), z(w, 4))
    with pytest.raises(ValueError, match="pages"):
        ParallelMixer(a(8), a(8))
    with pytest.raises(ValueError, match="width"):
        ParallelMixer(a(8), a(16))
    with pytest.raises(ValueError, match="rotation"):
        RotaryAttention(8, 1, 1, 4, 4, 1.0, z(12, 8), z(8, 4), rot_dims=4)


def test_random_weights_of_the_design():
    cfg = LirutarConfig.from_dict(LM.CFG_ALL)
    w = random_weights(lirutar_manifest(cfg), 3, is_norm=is_norm_weight)
    for name in ("embed.norm", "l0.norm1", "l1.norm2", "l0.mix.right.norm", "final.norm"):
        assert float(w[name].float().mean()) == 1.0, name
    for name in ("embed.norm.b", "l0.mix.left.q.b", "l0.mix.right.conv.b", "l1.mlp.correction"):
        assert abs(float(w[name].float().mean())) < 0.1, name


def test_frequencies_and_the_plain_pieces():
    assert np.allclose(_frequencies(10000.0, 8).numpy(), 10000.0 ** (-np.arange(4) / 4.0), rtol=1e-7)
    x = np.random.default_rng(0).standard_normal((3, 5, 12))
    y = PL.turn_halves(x, np.arange(5), 50.0, 8)
    assert np.array_equal(y[..., 8:], x[..., 8:]) and np.array_equal(y[:, 0], x[:, 0])
    assert np.allclose(y[:, 1, 1], x[:, 1, 1] * np.cos(50.0 ** -0.25) - x[:, 1, 5] * np.sin(50.0 ** -0.25))
    # a causal convolution: the last column meets the current token
    u = np.arange(1.0, 5.0)[:, None]
    assert np.allclose(PL.causal_conv(u, np.array([[100.0, 10.0, 1.0]]), np.array([0.5]))[:, 0], [1.5, 12.5, 123.5, 234.5])
    # parts of equal size, each by its own root mean square
    v = PL.rms_parts(np.array([3.0, 4.0, 0.0, 2.0]), 2, 0.0)
    assert np.allclose(v, [3 / 12.5 ** 0.5, 4 / 12.5 ** 0.5, 0.0, 2 ** 0.5])


def test_the_plain_router():
    r = dict(experts=4, identity=2, top=2, groups=dict(count=3, keep=1), scale=2.0)
    z = np.log(np.array([0.30, 0.05, 0.02, 0.28, 0.20, 0.15]))
    # without a correction the first group (best score 0.30) is kept: its two members, weighted by their own scores
    got = dict(PL.route(z, np.zeros(6), r))
    assert set(got) == {0, 1} and np.isclose(got[0], 2 * 0.30 / 0.35) and np.isclose(got[1], 2 * 0.05 / 0.35)
    # the correction moves the choice (every choice score may be negative), the weights stay the scores'
    got = dict(PL.route(z, np.array([-1.0, -1.0, -1.0, -1.0, -0.5, -0.9]), r))
    assert set(got) == {4, 5} and np.isclose(got[4], 2 * 0.20 / 0.35)
    # two groups kept: the largest of both
    got = PL.route(z, np.zeros(6), dict(r, groups=dict(count=3, keep=2)))
    assert [e for e, _ in got] == [0, 3]


def test_the_plain_recurrence_is_the_sum_over_earlier_tokens():
    """y_t = sum_(s <= t) prod_(s < r <= t) a_r dt_s (C_t . B_s) x_s + D x_t: the state written out."""
    cfg = LM.config(30, 16, [LM.layer(LM.att(1, 1, 4, 4, 0.5), LM.ssd(2, 3, 4, 1, 3, 2))])
    w = {k: v.astype(np.float64) for k, v in LM.make_tensors(cfg, 1).items()}
    h = np.random.default_rng(2).standard_normal((6, 16))
    m, p = cfg["layers"][0]["mixer"]["right"], "l0.mix.right."
    row = h @ w[p + "in"].T
    xbc = PL.silu(PL.causal_conv(row[:, 6:20], w[p + "conv"], w[p + "conv.b"]))
    x, B, C = xbc[:, :6].reshape(6, 2, 3), xbc[:, 6:10], xbc[:, 10:]
    dt = np.log1p(np.exp(row[:, 20:] + w[p + "dt_bias"]))
    a = np.exp(-np.exp(w[p + "A_log"]) * dt)
    y = w[p + "D"][None, :, None] * x
    for t in range(6):
        for s in range(t + 1):
            y[t] += (np.prod(a[s + 1:t + 1], axis=0) * dt[s] * (C[t] @ B[s]))[:, None] * x[s]
    g = y.reshape(6, 6) * row[:, :6] / (1 + np.exp(-row[:, :6]))
    want = (PL.rms_parts(g, 2, 1e-5) * w[p + "norm"]) @ w[p + "o"].T
    assert np.allclose(PL.ssd(w, p, m, h, 1e-5), want, rtol=1e-9, atol=1e-12)
