"""Lirutar through the engine against the plain implementation (tests/plain_lirutar.py), on small models of the tests' own.

Every comparison is between the engine's step function (cache and state manager, kernels, CUDA graphs as in serving) and
plain_lirutar.forward on whole sequences.  float32 is held to 1e-4 of the logits' scale; bfloat16 to what 8 bits of mantissa
cost on these sharp little models, by quantiles over the rows.
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_lirutar as PL
import replay_util as RU
import lirutar_models as LM

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
    cfg, W = PL.read_model(model_dir)
    return PL.forward(cfg, W, ids)


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
# each mechanism alone: models of one layer
# ---------------------------------------------------------------------------------------------------------------

_A, _S = LM.att(2, 1, 8, 8, 0.5), LM.ssd(2, 8, 8, 1, 2, 1)
_one = lambda left=_A, right=_S, mlp=None, ls=1.0, rs=1.0, loop=None: LM.config(40, 32, [LM.layer(left, right, mlp, ls, rs)], loop=loop)
ALONE = {
    "attention_bare": _one(rs=0.0),
    "attention_all_turned": _one(LM.att(2, 2, 16, 12, 0.3, (40.0, 16)), rs=0.0, ls=0.6),
    "attention_part_turned": _one(LM.att(6, 2, 24, 10, 0.25, (1000.0, 6)), rs=0.0, ls=1.7),
    "attention_window": _one(LM.att(3, 3, 8, 12, 0.6, (100.0, 4), 9), rs=0.0),
    "attention_window_one": _one(LM.att(4, 1, 8, 8, 0.6, (100.0, 8), 1), rs=0.0),
    "ssd": _one(right=LM.ssd(2, 16, 24, 1, 4, 2), ls=0.0),
    "ssd_groups": _one(right=LM.ssd(6, 8, 12, 3, 4, 6), ls=0.0, rs=0.4),
    "ssd_odd": _one(right=LM.ssd(3, 5, 37, 1, 3, 5), ls=0.0, rs=2.0),
    "ssd_one_tap": _one(right=LM.ssd(4, 8, 16, 4, 1, 1), ls=0.0),
    "ssd_six_taps": _one(right=LM.ssd(2, 8, 70, 2, 6, 1), ls=0.0),
    "ssd_wide_values": _one(right=LM.ssd(1, 72, 20, 1, 4, 9), ls=0.0),
    "both": _one(ls=0.3, rs=1.6),
    "dense_ff": _one(mlp=LM.dense(72)),
    "experts": _one(mlp=LM.moe(24, 0.7, 6, 2)),
    "experts_scaled_shared": _one(mlp=LM.moe(16, 1.5, 5, 3, scale=2.3, shared=(40, 0.6))),
    "experts_identities": _one(mlp=LM.moe(16, 1.0, 3, 2, identity=3)),
    "experts_groups": _one(mlp=LM.moe(8, 1.0, 6, 2, identity=2, count=4, keep=2)),
    "experts_all": _one(mlp=LM.moe(8, 1.0, 2, 3, identity=1)),
    "pass_once": _one(loop=(0, 1, 1)),
    "passes": _one(mlp=LM.dense(24), loop=(0, 1, 4)),
}


@pytest.mark.parametrize("name", sorted(ALONE))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_mechanism_alone(tmp_path, name, dtype):
    cfg = ALONE[name]
    d = LM.write_model(tmp_path / name, cfg, LM.make_tensors(cfg, 5))
    ids = _ids(np.random.default_rng(1), cfg["vocab"], 70)
    ref = _plain(d, ids)
    runner = _runner(d, dtype, tokens=128, page=8)
    whole = _play(runner, RU.whole("a", ids))
    one = _play(runner, RU.tail_one_by_one("b", ids, tail=69))        # the first token, then every token alone
    two = _play(runner, RU.changing_portions("c", ids, sizes=(2,)))   # portions of two
    for got, rid in ((whole, "a"), (one, "b"), (two, "c")):
        assert len(got) == len(ids)
        _close(got, {rid: ref}, dtype, rid)


def test_residual_stream_after_every_run(tmp_path):
    """The float32 engine's logits are right only if every run is; this pins which run of a layer a fault would be in."""
    from vitna_anchor_b200.engine.loading import load_model
    from vitna_anchor_b200.engine.runner import ModelRunner
    cj = LM.CONFIGS["all"]
    d = LM.make_model(tmp_path / "m", "all", seed=3)
    ids = _ids(np.random.default_rng(5), cj["vocab"], 40)
    cfg, W = PL.read_model(d)
    streams = []
    PL.forward(cfg, W, ids, layers_out=streams)
    model = load_model(d, "float32", "cuda")
    runner = ModelRunner(model, page_size=8, num_pages=8, max_requests=2, max_batch_tokens=64, max_model_len=64, cuda_graphs=False)
    runner.open("a")
    runner.cache.reserve_step([("a", len(ids))])
    ctx, rows = runner.builder.build([("a", ids, [])])
    seen = []
    ctx.after_run = lambda i: seen.append(ctx.workspace.rows("x", len(ids), cj["width"], torch.float32).cpu().numpy().copy())
    model.forward(ctx, rows)
    runner.cache.commit_step([("a", len(ids))])
    assert len(seen) == len(streams) == 8
    for i, (got, want) in enumerate(zip(seen, streams)):
        assert np.abs(got - want).max() < 2e-5 * max(1.0, np.abs(want).max()), i


# ---------------------------------------------------------------------------------------------------------------
# whole models: prompts, token by token, portions, mixed batches, pages and slots used again
# ---------------------------------------------------------------------------------------------------------------

@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("lirutar")
    out = {}
    for i, name in enumerate(sorted(LM.CONFIGS)):
        d = LM.make_model(root / name, name, seed=20 + i)
        rng = np.random.default_rng(200 + i)
        reqs = {f"r{k}": _ids(rng, LM.CONFIGS[name]["vocab"], n) for k, n in enumerate((150, 1, 37, 64, 91, 17))}
        out[name] = (d, reqs, {r: _plain(d, ids) for r, ids in reqs.items()})
    return out


@pytest.mark.parametrize("name", sorted(LM.CONFIGS))
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
    # portions of changing sizes down to two tokens, cut inside pages, windows and the convolution's reach
    runs["portions"] = {k: v for r, ids in reqs.items()
                        for k, v in _play(runner, RU.changing_portions(r, ids, sizes=(7, 2, 13, 3, 2, 29, 5, 2, 8, 11))).items()}
    # portions that end just before, at and just behind the end of a chunk of the recurrence
    runs["chunks"] = {k: v for r, ids in reqs.items() for k, v in _play(runner, RU.changing_portions(r, ids, sizes=(65, 63, 2, 64))).items()}
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


def test_a_request_alone_and_beside_others_on_other_pages_and_slots(models):
    """The same request first alone in a fresh engine, then as the fourth of four whose neighbours took the low pages and slots:
    its keys and its states (of every pass) sit elsewhere, and slots that others left are taken again."""
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
        assert np.abs(beside[k] - row).max() / np.abs(ref["r4"]).max() < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_slot_that_is_used_again_starts_from_nothing(models, dtype):
    """One state slot: every request takes the slot the one before it left, with that request's states and convolution inputs still in it."""
    d, reqs, ref = models["front"]
    runner = _runner(d, dtype, tokens=256, page=8, slots=1)
    for r in ("r0", "r2", "r1", "r5", "r2"):
        _close(_play(runner, RU.changing_portions(r, reqs[r], sizes=(5, 2, 31))), ref, dtype, r)


def test_a_step_that_fails_leaves_no_trace_in_any_pass(models):
    """A step given up in the second pass over the looped layers: the pages and the states of the passes that ran are put back."""
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
    """300 tokens one by one after a short prompt: the states are carried 300 times, the windows move 300 times, the rotations pass 300
    positions and the keys fill page after page while the windows' pages come back."""
    cfg = LM.CONFIGS["all"]
    d = LM.make_model(tmp_path / "m", "all", seed=77)
    ids = _ids(np.random.default_rng(8), cfg["vocab"], 310)
    ref = _plain(d, ids)
    for dtype in ("float32", "bfloat16"):
        got = _play(_runner(d, dtype, tokens=320, page=16), RU.tail_one_by_one("a", ids, tail=300))
        _close(got, {"a": ref}, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_state_that_hardly_decays_keeps_the_first_token(tmp_path, dtype):
    """Decays of nearly one, and a first token whose step size is a hundred times the others': after 400 tokens it still is most of the
    state.  A state that is lost, zeroed between steps or started late shows."""
    cfg = LM.config(50, 32, [LM.layer(LM.att(1, 1, 8, 8, 0.5), LM.ssd(2, 8, 8, 1, 2, 1), None, 0.0, 1.0)])
    t = LM.make_tensors(cfg, 4)
    p = "l0.mix.right."
    t[p + "A_log"][:] = -9.0
    t[p + "D"][:] = 0.0
    t[p + "dt_bias"][:] = -4.0
    t[p + "o"] *= 5.0
    t[p + "in"][-2:] = 0.0
    t[p + "in"][-2:, 0] = 2.0               # the step sizes read the first value, which only token 0's row has
    t["embed"][:, 0] = 0.0
    t["embed"][0, 0] = 20.0
    for n in ("embed.norm", "l0.norm1"):
        t[n][:], t[n + ".b"][:] = 1.0, 0.0
    d = LM.write_model(tmp_path / "m", cfg, t)
    ids = [0] + [int(v) for v in np.random.default_rng(9).integers(1, 50, 399)]
    c, W = PL.read_model(d)
    ref = PL.forward(c, W, ids)
    moved = PL.forward(c, W, [1] + ids[1:])[-1] - ref[-1]
    assert np.sqrt(np.mean(moved ** 2)) / np.sqrt(np.mean(ref ** 2)) > 0.15
    for steps in (RU.whole("a", ids), RU.changing_portions("a", ids, sizes=(100, 2, 1, 57)), RU.tail_one_by_one("a", ids, tail=399)):
        got = _play(_runner(d, dtype, tokens=512, page=16), steps)
        _close(got, {"a": ref}, dtype)
        _close({k: v for k, v in got.items() if k[1] == 399}, {"a": ref}, dtype)


# ---------------------------------------------------------------------------------------------------------------
# one key that must be found: far back, at the first positions, on either side of a page's border, on either side of a window's edge
# ---------------------------------------------------------------------------------------------------------------

def _needle(tmp_path, window=None, rotate=False, dim=32, vocab=1300):
    """One layer whose attention has one head (the other mixer's factor is 0).  A token's row has a key half and a value half; token t and
    token t + vocab / 2 share the key half and differ in the value half.  All norms have weight 1 and bias 0, queries and keys read the key
    half (W_q = W_k = [I 0], no bias) and values the value half, so a last token that is the partner of an earlier one gives half its
    weight to that one's value and half to its own, if and only if the earlier one is seen.  A wrong page, slot, offset or window shows."""
    width = 2 * dim
    cfg = LM.config(vocab, width, [LM.layer(LM.att(1, 1, dim, 24, 1.3, (10000.0, 4) if rotate else None, window), LM.ssd(1, 8, 8, 1, 2, 1), None, 1.0, 0.0)])
    t = LM.make_tensors(cfg, 6)
    rows = t["embed"].reshape(vocab, 2, dim)
    rows[vocab // 2:, 0] = rows[:vocab // 2, 0]
    rows -= rows.mean(axis=2, keepdims=True)            # every half has mean 0 and mean square 1: the norms leave it as it is
    t["embed"] = (rows / np.sqrt(np.mean(rows * rows, axis=2, keepdims=True))).reshape(vocab, width)
    for n in ("embed.norm", "l0.norm1"):
        t[n][:], t[n + ".b"][:] = 1.0, 0.0
    p = "l0.mix.left."
    half = np.concatenate([np.eye(dim), np.zeros((dim, dim))], axis=1).astype(np.float32)
    if rotate:              # the turned values weigh a quarter, so that a far key whose turn is opposite to the query's still has a share
        half[:4] *= 0.5
    for n in "qk":
        t[p + n], t[p + n + ".b"] = half.copy(), np.zeros(dim, dtype=np.float32)
    t[p + "v"][:, :dim] = 0.0
    t[p + "v"] *= 3.0
    return LM.write_model(tmp_path / f"needle{window}{rotate}", cfg, t, dtype=torch.float32), cfg


def _with_partner(base, place, vocab):
    return base[:-1] + [base[place] + vocab // 2]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rotate", [False, True])
def test_a_far_key_is_found_wherever_it_lies(tmp_path, dtype, rotate):
    d, cfg = _needle(tmp_path, rotate=rotate)
    n, page, V = 600, 16, cfg["vocab"]
    base = [int(t) for t in np.random.default_rng(0).permutation(V // 2)[:n]]           # all different
    c, W = PL.read_model(d)
    runner = _runner(d, dtype, tokens=640, page=page)
    for place in (0, 1, 3, page - 1, page, page + 1, 63, 64, 127, 128, 255, 256, 257, n - 3):
        ids = _with_partner(base, place, V)
        ref = PL.forward(c, W, ids)
        other = list(ids)
        other[place] = next(t for t in range(V // 2) if t not in base)
        moved = PL.forward(c, W, other)[-1] - ref[-1]
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
    c, W = PL.read_model(d)
    runner = _runner(d, dtype, tokens=384, page=page)
    for back in sorted({1, window - 2, window - 1, window, window + 1, 2 * window}):
        place = n - 1 - back
        ids = _with_partner(base, place, V)                              # the last token is the partner of the one at `place`
        ref = PL.forward(c, W, ids)
        other = list(ids)
        other[place] = next(t for t in range(V // 2) if t not in base)
        moved = PL.forward(c, W, other)[-1] - ref[-1]
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

SSD_SIZES = [(4, 2, 48, 24, 4), (3, 3, 5, 7, 3), (2, 1, 130, 72, 4), (6, 2, 64, 64, 2), (1, 1, 256, 16, 1), (4, 1, 16, 130, 7), (2, 2, 128, 63, 4)]


@pytest.mark.parametrize("sizes", SSD_SIZES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_recurrence_alone_in_its_forms(sizes, dtype):
    """ssd's kernels against the recurrence written out, on scattered slots over carried steps with a slot nobody holds: segments that
    end before, at and behind the end of a chunk, single tokens beside them, then steps of single tokens alone.  float32: token after
    token, and the one-launch form for single tokens; bfloat16: in chunks and the one-launch form, against token after token too.  The output
    goes into columns of a wider matrix."""
    from types import SimpleNamespace
    from vitna_anchor_b200 import ops
    H, G, N, P, taps = sizes
    rng = np.random.default_rng(N * 7 + P)
    inner, C, slots, off, eps, mult = H * P, H * P + 2 * G * N, 6, 3, 1e-5, 0.7
    width = off + inner + C + H + 2
    parts = next(p for p in (8, 3, 2, 1) if inner % p == 0)
    conv, conv_b = rng.standard_normal((C, taps)) * 0.6, rng.standard_normal(C) * 0.2
    dtb, a_log, D, w = rng.standard_normal(H) - 1, rng.standard_normal(H), rng.standard_normal(H), 1 + 0.2 * rng.standard_normal(inner)
    dev = [_dev(v) for v in (conv, conv_b, dtb, a_log, D, w)]
    f = lambda t: t.cpu().numpy().astype(np.float64)
    conv, conv_b, dtb, a_log, D, w = (f(t) for t in dev)
    state = torch.zeros(slots, ops.ssd_state_floats(H, G, N, P, taps), device="cuda")
    S, mem = np.zeros((slots, H, N, P)), np.zeros((slots, taps - 1, C))
    for lens, seg_slots in (((7, 1, 40, 65), (3, 0, 5, 1)), ((64, 2, 63, 1), (5, -1, 3, 0)), ((1, 1, 1), (0, 3, -1)), ((2, 3, 130), (0, 1, 3)), ((1, 1), (3, 1))):
        T = sum(lens)
        starts = np.concatenate([[0], np.cumsum(lens)]).astype(np.int32)
        single = all(n == 1 for n in lens)
        ctx = SimpleNamespace(seg_starts=torch.from_numpy(starts).cuda(), seg_slots=torch.tensor(seg_slots, dtype=torch.int32, device="cuda"),
                              token_seg=torch.from_numpy(np.repeat(np.arange(len(lens)), lens).astype(np.int32)).cuda(), num_segments=len(lens), decode_only=single)
        proj = _dev(rng.standard_normal((T, width)))
        new = lambda: (torch.empty(T, C, dtype=dtype, device="cuda"), torch.empty(T, 2 * H, device="cuda"), torch.empty(T, inner, device="cuda"),
                       torch.zeros(T, inner + 5, dtype=dtype, device="cuda"))
        scratch = torch.empty(ops.ssd_chunked_scratch_bytes(T, len(lens), H, N, P), dtype=torch.uint8, device="cuda")

        def run(st, c, chunks):
            xbc, gates, y, wide = new()
            ops.ssd(proj, off, *dev, eps, parts, mult, c, st, xbc, gates, y, wide[:, 4:4 + inner], H, G, N, P, taps, chunk_scratch=scratch if chunks else None)
            torch.cuda.synchronize()
            assert bool((wide[:, :4] == 0).all()) and bool((wide[:, 4 + inner:] == 0).all())
            return y, wide[:, 4:4 + inner].float()

        before = state.clone()
        was = ops.set_float32_exact(False)
        try:
            y, out = run(state, ctx, True)
            plain_state = before.clone()
            y2, out2 = run(plain_state, SimpleNamespace(**{**vars(ctx), "decode_only": False}), False)      # token after token
        finally:
            ops.set_float32_exact(was)
        p = f(proj)
        z, xr, dt = p[:, off:off + inner], p[:, off + inner:off + inner + C], np.logaddexp(0.0, p[:, off + inner + C:off + inner + C + H] + dtb)
        want = np.zeros((T, H, P))
        for s, slot in enumerate(seg_slots):
            a, b = starts[s], starts[s + 1]
            seen = np.concatenate([mem[slot] if slot >= 0 else np.zeros((taps - 1, C)), xr[a:b]])
            c = sum(seen[j:j + b - a] * conv[:, j] for j in range(taps)) + conv_b
            c = c * PL.sigmoid(c)
            if dtype == torch.bfloat16:
                c = torch.from_numpy(c.astype(np.float32)).bfloat16().double().numpy()
            St = S[slot].copy() if slot >= 0 else np.zeros((H, N, P))
            for t in range(a, b):
                for h in range(H):
                    g = h // (H // G)
                    x, B, Cc = c[t - a, h * P:(h + 1) * P], c[t - a, inner + g * N:inner + (g + 1) * N], c[t - a, inner + (G + g) * N:inner + (G + g + 1) * N]
                    St[h] = np.exp(-np.exp(a_log[h]) * dt[t, h]) * St[h] + dt[t, h] * B[:, None] * x[None, :]
                    want[t, h] = St[h].T @ Cc + D[h] * x
            if slot >= 0:
                S[slot], mem[slot] = St, seen[len(seen) - (taps - 1):] if taps > 1 else mem[slot]
        # in bfloat16 a convolution's result may round the other way here and there (2^-8 of one value of x, B or C)
        tol = 3e-5 if dtype == torch.float32 else 1e-2
        scale = max(1.0, np.abs(want).max())
        assert np.abs(f(y).reshape(T, H, P) - want).max() < tol * scale, lens
        assert np.sqrt(np.mean((f(y).reshape(T, H, P) - want) ** 2)) < 0.02 * tol * scale + 2e-6 * scale, lens
        gated = PL.rms_parts(want.reshape(T, inner) * PL.silu(z), parts, eps) * w * mult
        assert np.abs(f(out) - gated).max() < (1e-4 if dtype == torch.float32 else 6e-2) * max(1.0, np.abs(gated).max()), lens
        got_S = f(state)[:, :H * N * P].reshape(S.shape)
        assert np.abs(got_S - S).max() < tol * max(1.0, np.abs(S).max()), lens
        if taps > 1:
            assert np.abs(f(state)[:, H * N * P:H * N * P + (taps - 1) * C].reshape(mem.shape) - mem).max() < 1e-6
        # the two forms saw the same rounded inputs: they differ by float32 sums alone
        assert float((y - y2).abs().max()) < 5e-5 * scale and float((state - plain_state).abs().max()) < 5e-5 * max(1.0, np.abs(S).max()), lens


@pytest.mark.parametrize("sizes", [(4, 1, 64, 64, 8, 21), (6, 2, 32, 96, 16, 0), (3, 3, 24, 40, 8, 70), (8, 2, 128, 128, 16, 100)])
def test_attention_into_columns_of_a_wider_matrix(sizes):
    """The attention kernels write rows that lie apart; what they write is bit for bit what they write into a matrix of their own."""
    from types import SimpleNamespace
    from vitna_anchor_b200 import ops
    from vitna_anchor_b200.parts.base import GroupMeta, Workspace
    nh, nkv, hd, vd, ps, window = sizes
    rng = np.random.default_rng(hd + vd)
    ctx_len, lens = (200, 90, 150), (60, 1, 1)
    blocks = -(-max(ctx_len) // ps)
    bt = torch.from_numpy(rng.permutation(3 * blocks).reshape(3, blocks).astype(np.int32)).cuda()
    T = sum(lens)
    seg = torch.from_numpy(np.repeat(np.arange(3), lens).astype(np.int32)).cuda()
    pos = torch.from_numpy(np.concatenate([np.arange(c - n, c) for c, n in zip(ctx_len, lens)]).astype(np.int32)).cuda()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    for dtype in (torch.float32, torch.bfloat16):
        q, pages = _dev(rng.standard_normal((T, nh * hd)), dtype), _dev(rng.standard_normal((3 * blocks, ps * nkv * (hd + vd))), dtype)
        ctx = SimpleNamespace(num_dec=2, num_pre=60, token_seg=seg, positions=pos, dec_tokens=i32([60, 61]), pre_tokens=i32(list(range(60))),
                              pre_tiles=i32([[0, 60, 140, 0]]), max_context=200, workspace=Workspace(torch.device("cuda"), 128, 4, 256))
        meta = GroupMeta(None, bt, blocks)
        args = (q, pages, meta, ctx)
        was = ops.set_float32_exact(False)
        try:
            own = ops.attention_biased(*args, torch.empty(T, nh * vd, dtype=dtype, device="cuda"), nh, nkv, hd, vd, ps, hd ** -0.5, window)
            wide = torch.zeros(T, nh * vd + 24, dtype=dtype, device="cuda")
            ops.attention_biased(*args, wide[:, 8:8 + nh * vd], nh, nkv, hd, vd, ps, hd ** -0.5, window)
        finally:
            ops.set_float32_exact(was)
        assert torch.equal(wide[:, 8:8 + nh * vd], own)
        assert bool((wide[:, :8] == 0).all()) and bool((wide[:, 8 + nh * vd:] == 0).all())
        rows = ops.attention_rows_biased(q, pages, bt, seg, pos, torch.zeros(T, nh * vd + 8, dtype=dtype, device="cuda")[:, :nh * vd], nh, nkv, hd, vd, ps,
                                         hd ** -0.5, window)
        assert float((rows.float() - own.float()).abs().max()) < (2e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("case", [(8, 2, 2, 2, 1, 1.5), (6, 0, 3, 1, 1, 1.0), (20, 4, 5, 6, 2, 0.3), (60, 4, 8, 16, 3, 2.0), (4, 3, 4, 7, 6, 1.0)])
def test_the_scored_router_alone(case):
    from vitna_anchor_b200 import ops
    experts, identity, top, count, keep, scale = case
    rng = np.random.default_rng(experts)
    every, W = experts + identity, 40
    wr, corr = rng.standard_normal((every, W)) * 0.4, rng.standard_normal(every) * 0.3 - 0.4        # choice scores of both signs
    r = dict(experts=experts, top=top, groups=dict(count=count, keep=keep), scale=scale)
    for T in (1, 5, 130):
        x0 = rng.standard_normal((T, W))
        for dtype in (torch.float32, torch.bfloat16):
            x = _dev(x0, dtype)
            ids, wts = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
            ops.experts_route_scored(x, _dev(wr), _dev(corr), top, count, keep, scale, ids, wts)
            z = x.float().cpu().numpy().astype(np.float64) @ wr.astype(np.float32).T.astype(np.float64)
            for t in range(T):
                want = PL.route(z[t], corr.astype(np.float32).astype(np.float64), r)
                assert [int(e) for e in ids[t]] == [e for e, _ in want], (T, t)
                assert np.allclose(wts[t].cpu().numpy(), [v for _, v in want], rtol=2e-5, atol=1e-7)
    # equal choice scores: the lower index, in groups and among experts
    ids, wts = torch.empty(1, top, dtype=torch.int32, device="cuda"), torch.empty(1, top, device="cuda")
    ops.experts_route_scored(_dev(np.zeros((1, W))), _dev(wr), None, top, count, keep, scale, ids, wts)
    assert [int(e) for e in ids[0]] == list(range(top)) and np.allclose(wts.cpu().numpy(), scale / top, rtol=1e-5)


@pytest.mark.parametrize("T", [3, 40, 300])
def test_identities_in_both_forms_of_the_experts(T):
    """Ids of E and more take the token's input row: in the kernels that read an expert's rows for every pair and in the grouped products."""
    from vitna_anchor_b200 import ops
    rng = np.random.default_rng(T)
    E, W, ff, top, limit = 5, 64, 48, 3, 1.1
    gu, down, x = (_dev(rng.standard_normal(s) * sc, torch.bfloat16) for s, sc in (((E, 2 * ff, W), 0.2), ((E, W, ff), 0.15), ((T, W), 1.0)))
    ids = torch.from_numpy(np.stack([rng.permutation(E + 3)[:top] for _ in range(T)]).astype(np.int32)).cuda()
    wts = _dev(rng.random((T, top)))
    f = lambda t: t.float().cpu().numpy().astype(np.float64)
    want = np.zeros((T, W))
    for t in range(T):
        for k in range(top):
            e = int(ids[t, k])
            if e >= E:
                want[t] += f(wts)[t, k] * f(x)[t]
                continue
            h = f(gu)[e] @ f(x)[t]
            g, u = np.minimum(h[:ff], limit), np.clip(h[ff:], -limit, limit)
            want[t] += f(wts)[t, k] * (f(down)[e] @ (g * PL.sigmoid(1.702 * g) * (u + 1)))
    y = torch.zeros(T, W, device="cuda")
    ops.experts_apply(x, gu, down, ids, wts, torch.empty(T * top, ff, dtype=torch.bfloat16, device="cuda"), y, "clamped", limit)
    assert np.abs(f(y) - want).max() < 2e-2 * np.abs(want).max()
    rows = ops.experts_grouped_rows(T, top, E)
    new = lambda *s, dt=torch.bfloat16: torch.zeros(*s, dtype=dt, device="cuda")
    y2 = torch.zeros(T, W, device="cuda")
    ops.experts_apply_grouped(x, gu, down, ids, wts, new(T, top, dt=torch.int32), new(rows, dt=torch.int32), new(rows // 128, dt=torch.int32), new(rows, W),
                              new(rows, ff), new(rows, W, dt=torch.float32), y2, "clamped", limit, 1.702, new(rows, 2 * ff))
    assert np.abs(f(y2) - want).max() < 2e-2 * np.abs(want).max()


def test_the_pass_input_and_relu_squared():
    from vitna_anchor_b200 import ops
    rng = np.random.default_rng(3)
    for W in (32, 37):
        x, x0 = _dev(rng.standard_normal((9, W))), _dev(rng.standard_normal((9, W)))
        for dtype in (torch.float32, torch.bfloat16):
            cat = torch.empty(9, 2 * W, dtype=dtype, device="cuda")
            ops.pass_input(x0, cat, True, True)
            assert torch.equal(cat, torch.cat([x0, x0], dim=1).to(dtype))
            ops.pass_input(x, cat, True, False)
            assert torch.equal(cat, torch.cat([x, x0], dim=1).to(dtype))
    for (M, K, N) in ((3, 64, 96), (40, 96, 128), (200, 64, 512), (300, 512, 4096), (5, 36, 20)):       # few rows, the narrow and the wide tcgen05 product, odd
        for dtype in (torch.float32, torch.bfloat16):
            x, w = _dev(rng.standard_normal((M, K)), dtype), _dev(rng.standard_normal((N, K)) * K ** -0.5, dtype)
            got = ops.linear_act(x, w, torch.empty(M, N, dtype=dtype, device="cuda"), "relu2").float().cpu().numpy()
            want = np.maximum(x.float().cpu().numpy().astype(np.float64) @ w.float().cpu().numpy().astype(np.float64).T, 0.0) ** 2
            assert np.abs(got - want).max() < (1e-5 if dtype == torch.float32 else 1.2e-2) * np.abs(want).max(), (M, K, N, dtype)
    ops.check_device_errors()
    with pytest.raises(ops.KernelError, match="relu2"):
        ops.linear_gated(_dev(np.ones((2, 32))), _dev(np.ones((16, 32))), _dev(np.ones((2, 16))), _dev(np.ones((2, 8))), "relu2")


# ---------------------------------------------------------------------------------------------------------------
# the engine's own entry point and scheduler, the command line, the replay program
# ---------------------------------------------------------------------------------------------------------------

def _plain_greedy(model_dir, ids, n):
    cfg, W = PL.read_model(model_dir)
    ids = list(ids)
    for _ in range(n):
        ids.append(int(np.argmax(PL.forward(cfg, W, ids)[-1])))
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
    got = rp.run(RU.changing_portions("a", reqs["r4"]) + RU.tail_one_by_one("b", reqs["r2"], tail=10), LM.CONFIGS["wide"]["vocab"])
    rp.close()
    assert _worst(got, {"a": ref["r4"], "b": ref["r2"]}) < F32_TOL
    out = subprocess.run([sys.executable, os.path.join(RU.ROOT, "bin", "vitna-anchor"), "generate", "--model", d, "--ids",
                          ",".join(map(str, reqs["r5"])), "--max-new", "8", "--greedy", "--dtype", "float32"], capture_output=True, text=True)
    assert out.returncode == 0, out.stderr
    assert _plain_greedy(d, reqs["r5"], 8) == [int(t) for t in json.loads(out.stdout.strip().splitlines()[-1])["ids"]]
