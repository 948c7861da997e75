"""Zolapel through the engine against the plain implementation (tests/plain_zolapel.py), on small models of the tests' own.

Every comparison is between the engine's step function (cache and state manager, kernels, CUDA graphs as in serving) and
plain_zolapel.forward on whole sequences.  float32 is held to 1e-4 of the logits' scale; bfloat16 to what 8 bits of mantissa
cost on these sharp little models, by quantiles over the rows.
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_zolapel as PZ
import replay_util as RU
import zolapel_models as ZM

pytestmark = pytest.mark.gpu

F32_TOL = 1e-4
BF16_TOL = 1e-1                 # one row of a model that was made to be sharp at that row
BF16_MEDIAN, BF16_P90, BF16_WORST = 0.05, 0.2, 1.0       # the worst rows: a router's close call that went the other way


def _runner(model_dir, dtype, *, tokens=1024, page=16, slots=4, graphs=True):
    from vitna_anchor_b200.engine.loading import load_model
    from vitna_anchor_b200.engine.runner import ModelRunner
    model = load_model(model_dir, dtype, "cuda")
    return ModelRunner(model, page_size=page, num_pages=-(-tokens // page), max_requests=slots, max_batch_tokens=tokens,
                       max_model_len=min(model.max_positions, tokens), device="cuda", cuda_graphs=graphs)


def _play(runner, steps):
    """steps as replay_util makes them -> {(request, position): logits row}; requests are opened at their first entry and closed
    when a step ends them."""
    from vitna_anchor_b200.engine.runner import StepEntry
    got, at = {}, {}
    for entries, end in steps:
        for rid, _, _ in entries:
            if not runner.cache.is_open(rid):
                runner.open(rid)
        logits = runner.step([StepEntry(rid, list(map(int, toks)), list(want)) for rid, toks, want in entries])
        host = None if logits is None else logits.cpu().numpy()
        runner.check(sync=True)
        r = 0
        for rid, toks, want in entries:
            base = at.get(rid, 0)
            for w in want:
                got[(rid, base + w)] = host[r].copy()
                r += 1
            at[rid] = base + len(toks)
        for rid in end:
            runner.close(rid)
            at.pop(rid, None)
        runner.cache.check()
    return got


def _plain(model_dir, ids):
    cfg, W = PZ.read_model(model_dir)
    return PZ.forward(cfg, W, ids)


def _worst(got, want_by_req, rms=False):
    worst = 0.0
    for (rid, pos), row in got.items():
        ref = want_by_req[rid]
        if rms:
            worst = max(worst, float(np.sqrt(np.mean((row - ref[pos]) ** 2)) / np.sqrt(np.mean(ref ** 2))))
        else:
            worst = max(worst, float(np.abs(row - ref[pos]).max() / max(1.0, np.abs(ref).max())))
    return worst


def _close(got, want_by_req, dtype, what=None):
    """float32: every row within F32_TOL.  bfloat16: the rows' errors within the quantiles above (one row: within BF16_TOL)."""
    if dtype == "float32":
        w = _worst(got, want_by_req)
        assert w < F32_TOL, (what, w)
        return
    errs = np.array([np.sqrt(np.mean((row - want_by_req[rid][pos]) ** 2)) / np.sqrt(np.mean(want_by_req[rid] ** 2)) for (rid, pos), row in got.items()])
    if len(errs) == 1:
        assert errs[0] < BF16_TOL, (what, errs[0])
        return
    q = (float(np.median(errs)), float(np.quantile(errs, 0.9)), float(errs.max()))
    assert q[0] < BF16_MEDIAN and q[1] < BF16_P90 and q[2] < BF16_WORST, (what, q)


def _ids(rng, vocab, n):
    return [int(t) for t in rng.integers(0, vocab, n)]


def _dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).to("cuda").to(dtype)


# ---------------------------------------------------------------------------------------------------------------
# each mechanism alone: models of one or two layers
# ---------------------------------------------------------------------------------------------------------------

_A = ZM.att(2, 1, 8, 0.5)
_one = lambda mixer=_A, mlp=None, loop=None, side=None, mult=None: ZM.config(40, 32, [ZM.layer(mixer, mlp)], loop=loop, side=side, mult=mult)
ALONE = {
    "attention_bare": _one(),
    "attention_every_head_its_key": _one(ZM.att(3, 3, 16, 0.3)),
    "attention_all_turned": _one(ZM.att(2, 2, 16, 0.3, (40.0, 16))),
    "attention_part_turned": _one(ZM.att(6, 2, 24, 0.25, (1000.0, 6)), mult=0.7),
    "attention_bands": _one(ZM.att(4, 1, 32, 0.2, (20000.0, 32), scaling=ZM.BANDS)),
    "attention_odd_head": _one(ZM.att(3, 1, 9, 0.4, (100.0, 4))),
    "attention_wide_head": _one(ZM.att(2, 1, 136, 0.1, (100.0, 136))),
    "attention_window": _one(ZM.att(3, 3, 8, 0.6, (100.0, 4), 9)),
    "attention_window_one": _one(ZM.att(4, 1, 8, 0.6, (100.0, 8), 1)),
    "experts": _one(mlp=ZM.moe(24, 6, 2)),
    "experts_one": _one(mlp=ZM.moe(16, 5, 1), mult=1.4),
    "experts_all": _one(mlp=ZM.moe(8, 3, 3)),
    "experts_single": _one(mlp=ZM.moe(40, 1, 1)),
    "side": _one(side=16),
    "side_odd": _one(side=7, mult=0.3),
    "side_of_two_layers": ZM.config(40, 36, [ZM.layer(_A), ZM.layer(_A, ZM.moe(8, 2, 1))], side=8),
    "side_and_experts": _one(mlp=ZM.moe(24, 4, 2), side=24, mult=0.5),
    "pass_once": _one(loop=(0, 1, 1)),
    "passes": _one(mlp=ZM.moe(16, 3, 1), loop=(0, 1, 4), side=8),
    "passes_of_the_last": ZM.config(40, 32, [ZM.layer(_A), ZM.layer(ZM.att(1, 1, 16, 0.4, (30.0, 8), 11))], loop=(1, 2, 3), mult=0.8),
}


@pytest.mark.parametrize("name", sorted(ALONE))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_mechanism_alone(tmp_path, name, dtype):
    cfg = ALONE[name]
    d = ZM.write_model(tmp_path / name, cfg, ZM.make_tensors(cfg, 5))
    ids = _ids(np.random.default_rng(1), cfg["vocab"], 70)
    ref = _plain(d, ids)
    runner = _runner(d, dtype, tokens=128, page=8)
    whole = _play(runner, RU.whole("a", ids))
    one = _play(runner, RU.tail_one_by_one("b", ids, tail=69))        # the first token, then every token alone
    two = _play(runner, RU.changing_portions("c", ids, sizes=(2,)))   # portions of two
    for got, rid in ((whole, "a"), (one, "b"), (two, "c")):
        assert len(got) == len(ids)
        _close(got, {rid: ref}, dtype, rid)


@pytest.mark.parametrize("name", ["all", "odd", "front"])
@pytest.mark.parametrize("tokens", [1, 40])
def test_residual_stream_after_every_run(tmp_path, name, tokens):
    """The residual rows after every run of a layer, in 32-bit and (few tokens: with the per-layer input in one kernel) in the serving routing of it."""
    from vitna_anchor_b200 import ops
    from vitna_anchor_b200.engine.loading import load_model
    from vitna_anchor_b200.engine.runner import ModelRunner
    cj = ZM.CONFIGS[name]
    d = ZM.make_model(tmp_path / "m", name, seed=3)
    ids = _ids(np.random.default_rng(5), cj["vocab"], tokens)
    cfg, W = PZ.read_model(d)
    streams = []
    PZ.forward(cfg, W, ids, layers_out=streams)
    for exact in (True, False):
        was = ops.set_float32_exact(exact)
        try:
            model = load_model(d, "float32", "cuda")
            runner = ModelRunner(model, page_size=8, num_pages=8, max_requests=2, max_batch_tokens=64, max_model_len=64, cuda_graphs=False)
            runner.open("a")
            runner.cache.reserve_step([("a", len(ids))])
            ctx, rows = runner.builder.build([("a", ids, [])])
            seen = []
            ctx.after_run = lambda i: seen.append(ctx.workspace.rows("x", len(ids), cj["width"], torch.float32).cpu().numpy().copy())
            model.forward(ctx, rows)
            runner.cache.commit_step([("a", len(ids))])
        finally:
            ops.set_float32_exact(was)
        assert len(seen) == len(streams) == len(PZ.runs(cfg))
        for i, (got, want) in enumerate(zip(seen, streams)):
            assert np.abs(got - want).max() < 3e-5 * max(1.0, np.abs(want).max()), (exact, i)


# ---------------------------------------------------------------------------------------------------------------
# whole models: prompts, token by token, portions, mixed batches, pages and slots used again
# ---------------------------------------------------------------------------------------------------------------

@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("zolapel")
    out = {}
    for i, name in enumerate(sorted(ZM.CONFIGS)):
        d = ZM.make_model(root / name, name, seed=20 + i)
        rng = np.random.default_rng(200 + i)
        reqs = {f"r{k}": _ids(rng, ZM.CONFIGS[name]["vocab"], n) for k, n in enumerate((150, 1, 37, 64, 91, 17))}
        out[name] = (d, reqs, {r: _plain(d, ids) for r, ids in reqs.items()})
    return out


@pytest.mark.parametrize("name", sorted(ZM.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompts_decoding_portions_and_mixed_batches(models, name, dtype):
    d, reqs, ref = models[name]
    runner = _runner(d, dtype, tokens=384, page=8, slots=4)
    whole = {}
    for r, ids in reqs.items():
        whole.update(_play(runner, RU.whole(r, ids)))
    _close(whole, ref, dtype, "whole")
    runs = {}
    # the last 40 tokens one by one (the one-token request is a prompt of one token)
    runs["decode"] = {k: v for r, ids in reqs.items() for k, v in _play(runner, RU.tail_one_by_one(r, ids, tail=40)).items()}
    # portions of changing sizes down to two tokens, cut inside pages and windows
    runs["portions"] = {k: v for r, ids in reqs.items()
                        for k, v in _play(runner, RU.changing_portions(r, ids, sizes=(7, 2, 13, 3, 2, 29, 5, 2, 8, 11))).items()}
    # portions that end just before, at and just behind 64 tokens (the prompt attention's tiles)
    runs["tiles"] = {k: v for r, ids in reqs.items() for k, v in _play(runner, RU.changing_portions(r, ids, sizes=(65, 63, 2, 64))).items()}
    # up to four requests live, portions of some beside single tokens of others; six requests through four slots and a pool that
    # holds fewer positions than the requests have in all
    runs["mixed"] = _play(runner, RU.mixed(reqs, {r: max(1, len(ids) - 20) for r, ids in reqs.items()}, np.random.default_rng(3), live_max=4))
    # one prompt in portions beside decoding requests
    runs["beside"] = _play(runner, RU.mixed(reqs, {r: len(ids) // 2 for r, ids in reqs.items()}, np.random.default_rng(4), live_max=3,
                                           portions=(2, 40), one_prompt_at_a_time=True))
    for how, got in runs.items():
        assert len(got) == sum(len(i) for i in reqs.values()), how
        _close(got, ref, dtype, how)
        # and against the same engine's whole prompts: the way a request is cut moves nothing but rounding
        _close(got, {r: np.stack([whole[(r, p)] for p in range(len(ids))]) for r, ids in reqs.items()}, dtype, (how, "cut"))
    runner.cache.check()
    assert all(f == p.num_pages for f, p in zip(runner.cache.free_pages(), runner.cache.tables.pools))     # every page came back


@pytest.mark.parametrize("name", ["all", "wide"])
def test_the_32_bit_logits_are_the_same_bits_however_a_request_is_cut(models, name):
    """The exact routing: one order of sums, whatever the step brings; the experts' forms for few and for many tokens give the same bits."""
    d, reqs, _ = models[name]
    runner = _runner(d, "float32", tokens=384, page=8, slots=4)
    ids = reqs["r0"]
    whole = _play(runner, RU.whole("a", ids))
    for steps in (RU.tail_one_by_one("a", ids, tail=60), RU.changing_portions("a", ids, sizes=(3, 40, 2, 17))):
        got = _play(runner, steps)
        assert all(np.array_equal(got[k], whole[k]) for k in whole)
    mixed = _play(runner, RU.mixed({"a": ids, "b": reqs["r3"], "c": reqs["r4"]}, {"a": 120, "b": 30, "c": 60}, np.random.default_rng(1)))
    assert all(np.array_equal(mixed[k], whole[k]) for k in whole)


def test_a_request_alone_and_beside_others_on_other_pages_and_slots(models):
    """The same request first alone in a fresh engine, then as the fourth of four whose neighbours took the low pages and slots."""
    d, reqs, ref = models["all"]
    ids = reqs["r4"]
    alone = _play(_runner(d, "float32", tokens=512, page=8), RU.changing_portions("x", ids))
    runner = _runner(d, "float32", tokens=512, page=8)
    steps = [([("n0", reqs["r0"][:50], []), ("n1", reqs["r2"], []), ("n2", reqs["r3"][:9], [])], ["n1"])]      # n1's slot and pages come back
    steps += [([("n0", reqs["r0"][50:52], []), ("x", ids[:30], range(30)), ("n2", reqs["r3"][9:10], [])], [])]
    steps += [([("x", ids[30:31], [0]), ("n3", reqs["r5"], []), ("n0", reqs["r0"][52:53], [])], ["n3"])]
    steps += [([("x", ids[31:], range(len(ids) - 31)), ("n2", reqs["r3"][10:11], [])], ["x", "n0", "n2"])]
    beside = _play(runner, steps)
    for k, row in alone.items():
        assert np.array_equal(beside[k], row)


def test_a_step_that_fails_leaves_no_trace_in_any_pass(models):
    """A step given up in the second pass over the looped layers: the pages of the passes that ran are put back, and what a block left for the
    next one is nobody's."""
    from vitna_anchor_b200.engine.runner import StepEntry, StepFailed
    d, reqs, ref = models["all"]
    ids = reqs["r4"]
    runner = _runner(d, "float32", tokens=256, page=8)
    runner.open("a")
    runner.step([StepEntry("a", ids[:50], [])])
    for run, portion in ((4, ids[50:60]), (2, ids[50:51])):
        runner.fail_after_run_once(run)
        with pytest.raises(StepFailed):
            runner.step([StepEntry("a", portion, [])])
    got = runner.step([StepEntry("a", ids[50:], list(range(len(ids) - 50)))]).cpu().numpy()
    assert np.abs(got - ref["r4"][50:]).max() < F32_TOL * max(1.0, np.abs(ref["r4"]).max())


def test_long_decoding(tmp_path):
    """300 tokens one by one after a short prompt: the windows move 300 times, the rotations pass 300 positions and the keys fill page after
    page while the windows' pages come back."""
    cfg = ZM.CONFIGS["all"]
    d = ZM.make_model(tmp_path / "m", "all", seed=77)
    ids = _ids(np.random.default_rng(8), cfg["vocab"], 310)
    ref = _plain(d, ids)
    for dtype in ("float32", "bfloat16"):
        got = _play(_runner(d, dtype, tokens=320, page=16), RU.tail_one_by_one("a", ids, tail=300))
        _close(got, {"a": ref}, dtype)


def test_a_prompt_long_enough_for_the_grouped_products(tmp_path):
    """700 tokens whose experts run as products of row groups (the wide ones among them), then decoded tokens that read the same experts' rows."""
    cfg = ZM.config(90, 512, [ZM.layer(ZM.att(4, 2, 32, 0.2, (1000.0, 32), 100), ZM.moe(512, 12, 4)), ZM.layer(ZM.att(2, 1, 64, 0.1), ZM.moe(1024, 16, 6))],
                    loop=(0, 1, 2), side=64, mult=0.7)
    d = ZM.write_model(tmp_path / "m", cfg, ZM.make_tensors(cfg, 9))
    ids = _ids(np.random.default_rng(9), 90, 700)
    ref = _plain(d, ids)
    got = _play(_runner(d, "bfloat16", tokens=704, page=16), RU.tail_one_by_one("a", ids, tail=12))
    _close(got, {"a": ref}, "bfloat16")


# ---------------------------------------------------------------------------------------------------------------
# one key that must be found: far back, at the first positions, on either side of a page's border, on either side of a window's edge
# ---------------------------------------------------------------------------------------------------------------

def _needle(tmp_path, window=None, rotate=False, half=32, vocab=1300):
    """One layer with one head.  A token's row has a key half and a value half; token t and token t + vocab / 2 share the key half and differ in the
    value half.  Layer norms have weight 1 and bias 0 and leave the rows as they are.  A projected key is the whole row (and the value is it, as it
    is projected), a query the key half alone, so a last token that is the partner of an earlier one gives half its weight to that one's
    row and half to its own, if and only if the earlier one is seen.  A wrong page, slot, offset or window shows."""
    width = 2 * half
    cfg = ZM.config(vocab, width, [ZM.layer(ZM.att(1, 1, width, 0.4, (10000.0, 4) if rotate else None, window))])
    t = ZM.make_tensors(cfg, 6)
    rows = t["embed"].reshape(vocab, 2, half)
    rows[vocab // 2:, 0] = rows[:vocab // 2, 0]
    rows -= rows.mean(axis=2, keepdims=True)            # every half has mean 0 and mean square 1: the norms leave it as it is
    t["embed"] = (rows / np.sqrt(np.mean(rows * rows, axis=2, keepdims=True))).reshape(vocab, width)
    t["l0.norm1"][:], t["l0.norm1.b"][:] = 1.0, 0.0
    p = "l0.mix."
    t[p + "q.norm"][:], t[p + "k.norm"][:] = 1.0, 1.0
    if rotate:              # the turned values weigh a quarter, so that a far key whose turn is opposite to the query's still has a share
        t[p + "q.norm"][:4], t[p + "k.norm"][:4] = 0.5, 0.5
    t[p + "k"] = np.eye(width, dtype=np.float32)
    t[p + "q"] = np.concatenate([np.eye(width, dtype=np.float32)[:half], np.zeros((half, width), dtype=np.float32)])
    t[p + "g"] *= 0.2                    # a gate near a half for every token
    t["l0.ls1"] = np.full(width, 3.0, dtype=np.float32)
    return ZM.write_model(tmp_path / f"needle{window}{rotate}", cfg, t, dtype=torch.float32), cfg


def _with_partner(base, place, vocab):
    return base[:-1] + [base[place] + vocab // 2]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rotate", [False, True])
def test_a_far_key_is_found_wherever_it_lies(tmp_path, dtype, rotate):
    d, cfg = _needle(tmp_path, rotate=rotate)
    n, page, V = 600, 16, cfg["vocab"]
    base = [int(t) for t in np.random.default_rng(0).permutation(V // 2)[:n]]           # all different
    c, W = PZ.read_model(d)
    runner = _runner(d, dtype, tokens=640, page=page)
    for place in (0, 1, 3, page - 1, page, page + 1, 63, 64, 127, 128, 255, 256, 257, n - 3):
        ids = _with_partner(base, place, V)
        ref = PZ.forward(c, W, ids)
        other = list(ids)
        other[place] = next(t for t in range(V // 2) if t not in base)
        moved = PZ.forward(c, W, other)[-1] - ref[-1]
        assert np.sqrt(np.mean(moved ** 2)) / np.sqrt(np.mean(ref ** 2)) > 300 * F32_TOL, place
        for how, steps in (("prompt", RU.whole("a", ids)), ("decoded", RU.tail_one_by_one("a", ids, tail=2)),
                           ("portions", RU.changing_portions("a", ids, sizes=(250, 5, 2, 100)))):
            got = _play(runner, steps)
            _close({k: v for k, v in got.items() if k[1] == n - 1}, {"a": ref}, dtype, (place, how))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [3, 16, 41, 129])
def test_a_key_just_inside_and_just_outside_the_window(tmp_path, dtype, window):
    d, cfg = _needle(tmp_path, window=window, rotate=True)
    n, page, V = 300, 8, cfg["vocab"]
    base = [int(t) for t in np.random.default_rng(1).permutation(V // 2)[:n]]
    c, W = PZ.read_model(d)
    runner = _runner(d, dtype, tokens=384, page=page)
    for back in sorted({1, window - 2, window - 1, window, window + 1, 2 * window}):
        place = n - 1 - back
        ids = _with_partner(base, place, V)                              # the last token is the partner of the one at `place`
        ref = PZ.forward(c, W, ids)
        other = list(ids)
        other[place] = next(t for t in range(V // 2) if t not in base)
        moved = PZ.forward(c, W, other)[-1] - ref[-1]
        share = np.sqrt(np.mean(moved ** 2)) / np.sqrt(np.mean(ref ** 2))
        if back < window:
            assert share > 100 * F32_TOL, back                          # the last position that is seen: i - j = window - 1
        else:
            assert share == 0.0, back                                    # the first that is not
        for how, steps in (("prompt", RU.whole("a", ids)), ("decoded", RU.tail_one_by_one("a", ids, tail=max(2, min(back, 60) + 3))),
                           ("portions", RU.changing_portions("a", ids, sizes=(100, 5, 2, 37, 3)))):
            got = _play(runner, steps)
            _close({k: v for k, v in got.items() if k[1] == n - 1}, {"a": ref}, dtype, (back, how))
    runner.cache.check()


# ---------------------------------------------------------------------------------------------------------------
# kernels alone
# ---------------------------------------------------------------------------------------------------------------

_f = lambda t: t.float().cpu().numpy().astype(np.float64)


def _step_numpy(x, y, c, z, wz, mult, e, add, norm, eps):
    x = x.copy()
    if c is not None:
        x += c * y
    if z is not None:
        x += mult * PZ.rms(z, eps) * wz
    if e is not None:
        x += e
    if add is not None:
        x += add
    return x, (x if norm is None else PZ.layer_norm(x, norm[0], norm[1], eps))


@pytest.mark.parametrize("n", [32, 37, 576, 2048, 3000, 4096, 4100])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_step_between_sublayers_in_its_forms(n, dtype):
    from vitna_anchor_b200 import ops
    rng = np.random.default_rng(n)
    T, V, eps = 5, 11, 1e-5
    c, wz, add, wn, bn = (_dev(rng.standard_normal(n)) for _ in range(5))
    table, ids = _dev(rng.standard_normal((V, n)), dtype), torch.tensor([3, 0, 10, 3, 7], dtype=torch.int32, device="cuda")
    for bits in range(64):
        with_c, with_z, with_e, with_add, with_norm, with_out = (bool(bits >> k & 1) for k in range(6))
        if with_norm and not with_out:
            continue
        x, y, z = (_dev(rng.standard_normal((T, n))) for _ in range(3))
        out = torch.empty(T, n, dtype=dtype, device="cuda") if with_out else None
        want, normed = _step_numpy(_f(x), _f(y), _f(c) if with_c else None, _f(z) if with_z else None, _f(wz), 0.7, _f(table)[ids.cpu().numpy()] if with_e else None,
                                   _f(add) if with_add else None, (_f(wn), _f(bn)) if with_norm else None, eps)
        ops.residual_step(x, y, c if with_c else None, z=z if with_z else None, z_norm=wz, mult=0.7, table=table if with_e else None, ids=ids,
                          add=add if with_add else None, norm=(wn, bn) if with_norm else None, out=out, eps=eps)
        assert np.abs(_f(x) - want).max() < 2e-5 and not bool(y.any()), bits
        if with_out:
            assert np.abs(_f(out) - normed).max() < (3e-5 if dtype == torch.float32 else 2e-2) * max(1.0, np.abs(normed).max()), bits


@pytest.mark.parametrize("sizes", [(64, 12), (42, 5), (96, 16), (2048, 256), (1024, 128), (100, 64), (8, 3), (4000, 40)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_per_layer_input_in_one_kernel(sizes, dtype):
    from vitna_anchor_b200 import ops
    n, dim = sizes
    rng = np.random.default_rng(n + dim)
    V, off, eps, mult = 13, 3, 1e-5, 0.6
    gate, proj = _dev(rng.standard_normal((dim, n)) * n ** -0.5, dtype), _dev(rng.standard_normal((n, dim)), dtype)
    side, table = _dev(rng.standard_normal((V, dim + 9)), dtype), _dev(rng.standard_normal((V, n)), dtype)
    c, wz, add, wn, bn = (_dev(rng.standard_normal(n)) for _ in range(5))
    for T in (1, 3, 32):
        ids = torch.from_numpy(rng.integers(0, V, T).astype(np.int32)).cuda()
        rows = ids.cpu().numpy()
        for bits in range(16):
            with_c, with_e, with_add, with_norm = (bool(bits >> k & 1) for k in range(4))
            x, y = _dev(rng.standard_normal((T, n))), _dev(rng.standard_normal((T, n)))
            first = _f(x) + (_f(c) * _f(y) if with_c else 0.0)
            z = (PZ.gelu_tanh(first @ _f(gate).T) * _f(side)[rows, off:off + dim]) @ _f(proj).T
            want, normed = _step_numpy(_f(x), _f(y), _f(c) if with_c else None, z, _f(wz), mult, _f(table)[rows] if with_e else None,
                                       _f(add) if with_add else None, (_f(wn), _f(bn)) if with_norm else None, eps)
            out = torch.empty(T, n, dtype=dtype, device="cuda") if with_norm else None
            ops.token_side(x, y, c if with_c else None, gate, proj, side, off, wz, ids, mult=mult, table=table if with_e else None, add=add if with_add else None,
                           norm=(wn, bn) if with_norm else None, out=out, eps=eps)
            assert np.abs(_f(x) - want).max() < 1e-4 and not bool(y.any()), (T, bits)
            if with_norm:
                assert np.abs(_f(out) - normed).max() < (2e-4 if dtype == torch.float32 else 2e-2) * max(1.0, np.abs(normed).max()), (T, bits)
    a = _dev(rng.standard_normal((40, dim)))
    ids = torch.from_numpy(rng.integers(0, V, 40).astype(np.int32)).cuda()
    got = ops.token_gate(a, side, off, ids, torch.empty(40, dim, dtype=dtype, device="cuda"))
    want = PZ.gelu_tanh(_f(a)) * _f(side)[ids.cpu().numpy(), off:off + dim]
    assert np.abs(_f(got) - want).max() < (1e-5 if dtype == torch.float32 else 1e-2) * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("sizes", [(64, 12, 9), (2048, 256, 0), (96, 5, 3), (1024, 40, 24), (72, 128, 8), (42, 16, 0)])
@pytest.mark.parametrize("T", [7, 64, 70, 300])
def test_a_product_with_the_gate_and_the_token_s_factor_behind_it(sizes, T):
    from vitna_anchor_b200 import ops
    n, dim, off = sizes
    rng = np.random.default_rng(n + T)
    V = 17
    for dtype in (torch.float32, torch.bfloat16):
        x, w = _dev(rng.standard_normal((T, n)), dtype), _dev(rng.standard_normal((dim, n)) * n ** -0.5, dtype)
        side = _dev(rng.standard_normal((V, dim + off + 8)), dtype)
        ids = torch.from_numpy(rng.integers(0, V, T).astype(np.int32)).cuda()
        out = torch.zeros(T, dim, dtype=dtype, device="cuda")
        ops.linear_token_gate(x, w, side, off, ids, torch.empty(T, dim, device="cuda"), out)
        want = PZ.gelu_tanh(_f(x) @ _f(w).T) * _f(side)[ids.cpu().numpy(), off:off + dim]
        assert np.abs(_f(out) - want).max() < (2e-5 if dtype == torch.float32 else 2e-2) * max(1.0, np.abs(want).max()), dtype
    ops.check_device_errors()


@pytest.mark.parametrize("sizes", [(4, 2, 16, 16, 8), (3, 1, 96, 96, 96), (20, 4, 64, 64, 30), (5, 5, 7, 7, 2), (2, 1, 256, 256, 256), (3, 3, 12, 20, 6), (2, 2, 260, 260, 8),
                                   (1, 1, 10, 10, 0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_heads_are_normed_turned_and_stored(sizes, dtype):
    """Norms or none, pairs of neighbours or of halves, values of their own or the projected keys; scattered slots, one token that is not written."""
    from vitna_anchor_b200 import ops
    H, G, hd, vd, dims = sizes
    rng = np.random.default_rng(hd * 3 + H)
    T, ps, pages, off, eps = 6, 4, 5, 2, 1e-5
    positions = torch.tensor([0, 1, 77, 4000, 123456, 9], dtype=torch.int32, device="cuda")
    slot = torch.tensor([3, 17, -1, 8, 0, 11], dtype=torch.int32, device="cuda")
    freq = _dev(PZ.frequencies(10000.0, dims)) if dims else None
    qn, kn = _dev(1 + 0.3 * rng.standard_normal(hd)), _dev(1 + 0.3 * rng.standard_normal(hd))
    for normed, neighbours, from_k in [(a, b, c) for a in (True, False) for b in (True, False) for c in (True, False)]:
        if from_k and vd != hd:
            continue
        cols = (H + G) * hd + (0 if from_k else G * vd)
        proj = _dev(rng.standard_normal((T, off + cols + 4)))
        cache = torch.zeros(pages, ps * G * (hd + vd), dtype=dtype, device="cuda")
        q = torch.zeros(T, H * hd, dtype=dtype, device="cuda")
        ops.mixed_attn_prepare(proj, positions, slot, qn if normed else None, kn if normed else None, eps if normed else -1.0, freq, dims, None, q, cache, H, G, hd, vd,
                               ps, off=off, neighbours=neighbours, v_from_k=from_k)
        p = _f(proj)[:, off:]
        heads = p[:, :(H + G) * hd].reshape(T, H + G, hd).transpose(1, 0, 2)
        v = heads[H:] if from_k else p[:, (H + G) * hd:(H + G) * hd + G * vd].reshape(T, G, vd).transpose(1, 0, 2)
        y = np.concatenate([PZ.rms(heads[:H], eps) * _f(qn), PZ.rms(heads[H:], eps) * _f(kn)]) if normed else heads
        if dims:
            ang = (np.float32(1) * positions.cpu().numpy().astype(np.float32)[:, None] * freq.cpu().numpy()[None, :]).astype(np.float64)
            c, s, half = np.cos(ang), np.sin(ang), dims // 2
            a, b = (slice(0, dims, 2), slice(1, dims, 2)) if neighbours else (slice(0, half), slice(half, dims))
            out = y.copy()
            out[..., a], out[..., b] = y[..., a] * c - y[..., b] * s, y[..., b] * c + y[..., a] * s
            y = out
        tol = (2e-5 if dtype == torch.float32 else 1.2e-2) * max(1.0, np.abs(y).max())
        what = (normed, neighbours, from_k)
        assert np.abs(_f(q).reshape(T, H, hd).transpose(1, 0, 2) - y[:H]).max() < tol, what
        ck = _f(cache)[:, :G * ps * hd].reshape(pages, G, ps, hd)
        cv = _f(cache)[:, G * ps * hd:].reshape(pages, G, ps, vd)
        written = np.zeros((pages, ps), dtype=bool)
        for t, s_ in enumerate(slot.cpu().numpy()):
            if s_ < 0:
                continue
            written[s_ // ps, s_ % ps] = True
            assert np.abs(ck[s_ // ps, :, s_ % ps] - y[H:, t]).max() < tol and np.abs(cv[s_ // ps, :, s_ % ps] - v[:, t]).max() < tol, (what, t)
        assert not ck.transpose(0, 2, 1, 3)[~written].any() and not cv.transpose(0, 2, 1, 3)[~written].any(), what


@pytest.mark.parametrize("sizes", [(4, 1, 64, 64, 8, 21), (6, 2, 32, 32, 16, 0), (3, 3, 24, 24, 8, 70), (8, 2, 128, 128, 16, 100), (16, 1, 96, 96, 16, 0), (40, 2, 64, 64, 16, 129)])
def test_a_gate_a_head_in_every_attention_kernel(sizes):
    """The gated output is the ungated one times the sigmoid, in the kernels for decoded tokens, prompt portions and all the rest."""
    from types import SimpleNamespace
    from vitna_anchor_b200 import ops
    from vitna_anchor_b200.parts.base import GroupMeta, Workspace
    nh, nkv, hd, vd, ps, window = sizes
    rng = np.random.default_rng(hd + nh)
    ctx_len, lens = (700, 90, 550), (60, 1, 1)
    blocks = -(-max(ctx_len) // ps)
    bt = torch.from_numpy(rng.permutation(3 * blocks).reshape(3, blocks).astype(np.int32)).cuda()
    T = sum(lens)
    seg = torch.from_numpy(np.repeat(np.arange(3), lens).astype(np.int32)).cuda()
    pos = torch.from_numpy(np.concatenate([np.arange(c - n, c) for c, n in zip(ctx_len, lens)]).astype(np.int32)).cuda()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    wide = _dev(2 * rng.standard_normal((T, nh + 7)))
    gate = wide[:, 3:3 + nh]
    factor = 1.0 / (1.0 + np.exp(-_f(gate)))
    for dtype in (torch.float32, torch.bfloat16):
        q, pages = _dev(rng.standard_normal((T, nh * hd)), dtype), _dev(rng.standard_normal((3 * blocks, ps * nkv * (hd + vd))), dtype)
        ctx = SimpleNamespace(num_dec=2, num_pre=60, token_seg=seg, positions=pos, dec_tokens=i32([60, 61]), pre_tokens=i32(list(range(60))),
                              pre_tiles=i32([[0, 60, 640, 0]]), max_context=700, workspace=Workspace(torch.device("cuda"), 128, 4, 1024))
        meta = GroupMeta(None, bt, blocks)
        new = lambda: torch.empty(T, nh * vd, dtype=dtype, device="cuda")
        tol = 1e-5 if dtype == torch.float32 else 2e-2
        for exact in (True, False):
            was = ops.set_float32_exact(exact)
            try:
                plain = ops.attention_biased(q, pages, meta, ctx, new(), nh, nkv, hd, vd, ps, hd ** -0.5, window)
                got = ops.attention_biased(q, pages, meta, ctx, new(), nh, nkv, hd, vd, ps, hd ** -0.5, window, gate=gate)
            finally:
                ops.set_float32_exact(was)
            want = (_f(plain).reshape(T, nh, vd) * factor[:, :, None]).reshape(T, nh * vd)
            assert np.abs(_f(got) - want).max() < tol * max(1.0, np.abs(want).max()), (dtype, exact)
    with pytest.raises(ops.KernelError, match="gate"):
        ops.attention_biased(q, pages, meta, ctx, new(), nh, nkv, hd, vd, ps, 1.0, window, gate=wide)


@pytest.mark.parametrize("case", [(16, 1), (8, 3), (5, 5), (70, 6), (1, 1)])
def test_the_router_with_a_sigmoid_for_every_score(case):
    from vitna_anchor_b200 import ops
    E, top = case
    rng = np.random.default_rng(E)
    W = 40
    wr, corr = _dev(rng.standard_normal((E, W)) * 0.4), _dev(rng.standard_normal(E) * 0.3)
    for T in (1, 5, 130):
        for dtype in (torch.float32, torch.bfloat16):
            x = _dev(rng.standard_normal((T, W)), dtype)
            s = PZ.sigmoid(_f(x) @ _f(wr).T)
            for c, squared, scale in ((None, False, 1.0), (None, True, 1.0), (corr, False, 1.7), (corr, True, 0.5)):
                ids, wts = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
                ops.experts_route_scored(x, wr, c, top, 1, 1, scale, ids, wts, True, squared)
                choice = s + (0.0 if c is None else _f(c))
                for t in range(T):
                    want = sorted(range(E), key=lambda e: -choice[t, e])[:top]
                    assert [int(e) for e in ids[t]] == want, (T, t)
                    w = s[t, want] * scale
                    assert np.allclose(_f(wts)[t], w * w if squared else w, rtol=2e-5, atol=1e-7)
    # scores that round to 1: the logits still tell the experts apart
    if E > 2 * top:
        big = _dev(20.0 + rng.permutation(E)[:, None] + np.zeros((E, W)))
        ids, wts = torch.empty(1, top, dtype=torch.int32, device="cuda"), torch.empty(1, top, device="cuda")
        ops.experts_route_scored(_dev(np.ones((1, W))), big, None, top, 1, 1, 1.0, ids, wts, True, False)
        assert [int(e) for e in ids[0]] == [int(e) for e in np.argsort(-_f(big)[:, 0])[:top]] and bool((wts == 1.0).all())


def _experts_numpy(x, w, down, ids, wts, activation, limit, E, gated):
    T, top = ids.shape
    want = np.zeros(x.shape)
    ff = down.shape[2]
    for t in range(T):
        for k in range(top):
            e = int(ids[t, k])
            if e >= E:
                want[t] += wts[t, k] * x[t]
                continue
            h = w[e] @ x[t]
            if not gated:
                a = np.maximum(h, 0.0) ** 2 if activation == "relu2" else PZ.gelu_tanh(h)
            elif activation == "clamped":
                g = np.minimum(h[:ff], limit)
                a = g * PZ.sigmoid(1.702 * g) * (np.clip(h[ff:], -limit, limit) + 1)
            else:
                a = h[:ff] * PZ.sigmoid(h[:ff]) * h[ff:]
            want[t] += wts[t, k] * (down[e] @ a)
    return want


@pytest.mark.parametrize("kind", ["relu2", "gelu_tanh", "silu", "clamped"])
@pytest.mark.parametrize("case", [(8, 1, 16, 64, 48, 0), (20, 4, 6, 96, 40, 2), (60, 3, 3, 64, 128, 0), (3, 2, 4, 512, 72, 0), (128, 2, 5, 48, 24, 1)])
def test_few_tokens_that_share_experts_give_the_same_bits(kind, case):
    """Every chosen expert's rows read once for all tokens that chose it, against the kernels that read them for every token: more pairs an expert than
    a pass takes, experts nobody chose, identities, one expert a token (added to y by the second kernel itself)."""
    from vitna_anchor_b200 import ops
    T, top, E, W, ff, identities = case
    gated = kind in ("silu", "clamped")
    rng = np.random.default_rng(T + ff)
    for dtype in (torch.float32, torch.bfloat16):
        w, down, x = (_dev(rng.standard_normal(s) * sc, dtype) for s, sc in (((E, (2 if gated else 1) * ff, W), W ** -0.5), ((E, W, ff), ff ** -0.5), ((T, W), 1.0)))
        ids = torch.from_numpy(np.stack([rng.permutation(E + identities)[:top] for _ in range(T)]).astype(np.int32)).cuda()
        if E > 4:
            ids[ids == 2] = 3 if top == 1 else 2
        wts = _dev(rng.random((T, top)))
        y0 = _dev(rng.standard_normal((T, W)))
        args = dict(activation=kind, limit=0.9, gated=gated)
        buf = lambda: torch.zeros(T * top, ff, dtype=dtype, device="cuda")
        y1, y2 = y0.clone(), y0.clone()
        a1, a2 = buf(), buf()
        ops.experts_apply(x, w, down, ids, wts, a1, y1, **args)
        ops.experts_apply_shared(x, w, down, ids, wts, a2, torch.empty(T * top, W, device="cuda"), y2, **args)
        assert torch.equal(a1, a2) and torch.equal(y1, y2)
        if top == 1 and not identities:
            y3 = y0.clone()
            ops.experts_apply_shared(x, w, down, ids, wts, buf(), None, y3, **args)
            assert torch.equal(y1, y3)
        want = _f(y0) + _experts_numpy(_f(x), _f(w), _f(down), ids.cpu().numpy(), _f(wts), kind, 0.9, E, gated)
        assert np.abs(_f(y1) - want).max() < (2e-5 if dtype == torch.float32 else 3e-2) * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("kind", ["relu2", "gelu_tanh", "silu", "clamped"])
@pytest.mark.parametrize("case", [(300, 2, 5, 64, 48), (700, 3, 9, 512, 512), (1500, 2, 4, 640, 1032)])
def test_the_grouped_products_gated_and_not(kind, case):
    """Row groups on the tensor cores, narrow tiles and wide ones, with an expert nobody chose, against the row-reading kernels."""
    from vitna_anchor_b200 import ops
    T, top, E, W, ff = case
    gated = kind in ("silu", "clamped")
    rng = np.random.default_rng(T)
    per = 2 if gated else 1
    bf = torch.bfloat16
    w, down, x = (_dev(rng.standard_normal(s) * sc, bf) for s, sc in (((E, per * ff, W), W ** -0.5), ((E, W, ff), ff ** -0.5), ((T, W), 1.0)))
    ids = torch.from_numpy(np.stack([rng.permutation(E - 1)[:top] for _ in range(T)]).astype(np.int32)).cuda()
    wts = _dev(rng.random((T, top)))
    y1, y2 = torch.zeros(T, W, device="cuda"), torch.zeros(T, W, device="cuda")
    ops.experts_apply(x, w, down, ids, wts, torch.zeros(T * top, ff, dtype=bf, device="cuda"), y1, kind, 0.9, 1.702, gated)
    rows = ops.experts_grouped_rows(T, top, E)
    new = lambda *s, dt=bf: torch.zeros(*s, dtype=dt, device="cuda")
    ops.experts_apply_grouped(x, w, down, ids, wts, new(T, top, dt=torch.int32), new(rows, dt=torch.int32), new(rows // 128, dt=torch.int32), new(rows, W),
                              new(rows, ff), new(rows, W, dt=torch.float32), y2, kind, 0.9, 1.702, new(rows, 2 * ff) if kind == "clamped" else None, gated)
    torch.cuda.synchronize()
    ops.check_device_errors()
    assert float((y1 - y2).abs().max()) < 2e-2 * float(y1.abs().max())


def test_what_a_pass_begins_with_deferred_and_not(models):
    """PassOffset in front of a block that takes it up in its first kernel, and as a launch of its own."""
    from types import SimpleNamespace
    from vitna_anchor_b200.parts.block import ScaledResidualBlock
    from vitna_anchor_b200.parts.loop import PassOffset
    rng = np.random.default_rng(1)
    for dtype in (torch.float32, torch.bfloat16):
        table, step, x = _dev(rng.standard_normal((9, 24)), dtype), _dev(rng.standard_normal(24)), _dev(rng.standard_normal((4, 24)))
        tokens = torch.tensor([8, 0, 3, 3], dtype=torch.int32, device="cuda")
        ctx = SimpleNamespace(tokens=tokens, extra={"pass": 1})
        for tb in (table, None):
            got = x.clone()
            PassOffset(24, step, tb).forward(got, ctx)
            want = _f(x) + _f(step) + (_f(table)[[8, 0, 3, 3]] if tb is not None else 0.0)
            assert np.abs(_f(got) - want).max() < 1e-6
            PassOffset(24, step, tb, deferred=True).forward(got, ctx)
            assert np.abs(_f(got) - want).max() < 1e-6 and ctx.extra[ScaledResidualBlock.ADDITION][1] is tb


# ---------------------------------------------------------------------------------------------------------------
# the engine's own entry point and scheduler, the command line, the replay program
# ---------------------------------------------------------------------------------------------------------------

def _plain_greedy(model_dir, ids, n):
    cfg, W = PZ.read_model(model_dir)
    ids = list(ids)
    for _ in range(n):
        ids.append(int(np.argmax(PZ.forward(cfg, W, ids)[-1])))
    return ids[-n:]


def test_greedy_generation_through_the_engine_and_its_scheduler(models):
    from vitna_anchor_b200.engine.engine import Engine
    d, reqs, _ = models["all"]
    eng = Engine(d, dtype="float32", parallel=3, kv_block=8, max_batch_tokens=64, max_prompt_portion=24)
    prompts = [reqs["r2"], reqs["r5"], reqs["r1"], reqs["r3"][:30]]       # four requests through three slots
    handles = [eng.add_request(p, max_new=12) for p in prompts]
    while eng.scheduler.has_work():
        eng.step()
    eng.flush()
    for h, p in zip(handles, prompts):
        assert list(h.output) == _plain_greedy(d, p, 12)
    assert eng.generate(prompts[0], max_new=12) == _plain_greedy(d, prompts[0], 12)


def test_the_replay_program_and_the_command_line(models, tmp_path):
    d, reqs, ref = models["wide"]
    rp = RU.Replay(d, "float32", tmp_path / "out", max_tokens=256, kv_block=8)
    got = rp.run(RU.changing_portions("a", reqs["r4"]) + RU.tail_one_by_one("b", reqs["r2"], tail=10), ZM.CONFIGS["wide"]["vocab"])
    rp.close()
    assert _worst(got, {"a": ref["r4"], "b": ref["r2"]}) < F32_TOL
    out = subprocess.run([sys.executable, os.path.join(RU.ROOT, "bin", "vitna-anchor"), "generate", "--model", d, "--ids",
                          ",".join(map(str, reqs["r5"])), "--max-new", "8", "--greedy", "--dtype", "float32"], capture_output=True, text=True)
    assert out.returncode == 0, out.stderr
    assert _plain_greedy(d, reqs["r5"], 8) == [int(t) for t in json.loads(out.stdout.strip().splitlines()[-1])["ids"]]
