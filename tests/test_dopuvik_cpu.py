"""Dopuvik without a GPU: its configuration, its tensor declarations, the plain implementation's
own mechanisms, and the engine's host side (pages of kept first tokens beside a window's, two
state records of one mixer, batch packing, step function) driven through the plain kernel
references against the plain implementation of the whole design."""
import math
import random

import numpy as np
import pytest
import torch

import dopuvik_tiny as dv
import plain_dopuvik as plain
import schedules
from plain_ops import PlainOps
from rvllm_b200.cache import CacheManager
from rvllm_b200.config import config_from_dict
from rvllm_b200.config.registry import architecture
from rvllm_b200.engine import ModelRunner, load_model, make_cache
from rvllm_b200.errors import ConfigError
from rvllm_b200.parts.base import PagedNeed, SeveralNeeds, StateNeed
from rvllm_b200.parts.model import param_decls


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = str(tmp_path_factory.mktemp("do"))
    return {n: dv.write(root, n) for n in dv.CONFIGS}


def test_config_round_trip_and_errors():
    for name in dv.CONFIGS:
        cfg = config_from_dict(dv.config(name))
        assert config_from_dict(cfg.to_dict()) == cfg
        assert cfg.architecture == "Dopuvik"

    def refused(change):
        bad = dv.config("A")
        change(bad)
        with pytest.raises(ConfigError):
            config_from_dict(bad)

    mixer = lambda c, i: c["layers"][i]["mixer"]
    router = lambda c: c["layers"][0]["mlp"]["router"]
    refused(lambda c: mixer(c, 0).update(groups=4))                     # does not divide the heads
    refused(lambda c: mixer(c, 0).update(norm_groups=7))                # no equal parts
    refused(lambda c: mixer(c, 1)["left"].update(kv_heads=4))
    refused(lambda c: mixer(c, 1)["right"].update(kv_heads=3))
    refused(lambda c: mixer(c, 1)["left"]["rot"].update(dims=34))       # more than a head has
    refused(lambda c: mixer(c, 1)["left"]["mask"].update(size=0))
    refused(lambda c: mixer(c, 1).pop("right"))
    refused(lambda c: mixer(c, 2)["rot"].update(dims=10))               # the whole part turns
    refused(lambda c: mixer(c, 2).pop("rot"))
    refused(lambda c: mixer(c, 2)["rot"]["scaling"].update(fast=0))
    refused(lambda c: router(c).update(identity=4))                     # no equal groups
    refused(lambda c: router(c).update(top=7))                          # more than the kept groups have
    refused(lambda c: router(c)["groups"].update(keep=6))
    refused(lambda c: c["layers"][0].update(type="sideways"))
    refused(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    refused(lambda c: c.pop("norm"))


def test_declared_tensors_and_constants():
    cfg = config_from_dict(dv.config("A"))
    spec = architecture("Dopuvik").build_spec(cfg)
    shapes = {n: d.shape for n, d in param_decls(spec).items()}
    assert shapes["embed"] == shapes["head"] == (300, 96) and shapes["final.norm"] == (96,)
    # z | x | B | C | dt
    assert shapes["l0.mix.in"] == (2 * 96 + 2 * 2 * 24 + 6, 96)
    assert shapes["l0.mix.conv"] == (96 + 96, 3) and shapes["l0.mix.conv.b"] == (192,)
    assert shapes["l0.mix.dt_bias"] == shapes["l0.mix.A_log"] == shapes["l0.mix.D"] == (6,)
    assert shapes["l0.mix.norm"] == (96,) and shapes["l0.mix.o"] == (96, 96)
    assert shapes["l0.mlp.router"] == (10, 96) and shapes["l0.mlp.correction"] == (10,)
    assert "l0.mlp.e6.gate" in shapes and "l0.mlp.e7.gate" not in shapes
    assert shapes["l1.mix.left.q"] == (192, 96) and shapes["l1.mix.left.q.b"] == (192,)
    assert shapes["l1.mix.left.v"] == (32, 96) and shapes["l1.mix.left.o"] == (96, 96)
    assert shapes["l1.mix.left.o.b"] == (96,)
    assert shapes["l1.mix.right.a"] == shapes["l1.mix.right.b"] == (4, 96)
    assert shapes["l1.mix.right.dt_bias"] == (4,) and shapes["l1.mix.right.g"] == (64, 96)
    assert shapes["l1.mix.right.k.conv"] == (48, 4) and shapes["l1.mix.right.norm"] == (16,)
    assert shapes["l2.mix.dkv"] == (60, 96) and shapes["l2.mix.uq"] == (4 * 36, 56)
    assert "l2.norm2" not in shapes and "l0.norm1.b" not in shapes
    assert spec.embedding_scale == 9.0 and spec.logit_scale == 0.3
    moe = spec.layers[0].feed_forward
    assert (moe.experts, moe.identity, moe.outputs, moe.groups, moe.keep, moe.group_top) == (7, 3, 10, 5, 3, 1)
    assert not moe.renormalize and moe.route_scale == 2.5 and moe.score == "softmax"
    left = spec.layers[1].mixer.branches[0]
    assert (left.window, left.keep_first) == (20, 7)


def test_what_a_call_remembers(folders):
    model, _ = load_model(folders["A"], "float32", "cpu", PlainOps())
    needs = model.cache_needs()
    assert needs[0] == SeveralNeeds((StateNeed((2, 192)), StateNeed((6 * 24 * 16,))))
    delta = 3 * (2 * 2 * 24 + 4 * 16) + 4 * 24 * 16
    assert needs[1] == SeveralNeeds((PagedNeed(2, 32, 20, v_head_dim=16, keep_first=7), StateNeed((delta,))))
    assert needs[2] == PagedNeed(1, 60, 13, values=False)
    model, _ = load_model(folders["C"], "float32", "cpu", PlainOps())
    assert model.cache_needs()[3] == SeveralNeeds((None, StateNeed((2 * 3 * 9,))))   # one tap: no inputs


# ---- the cache: first tokens that stay -------------------------------------------------------

@pytest.mark.parametrize("window,keep,page", [(8, 3, 2), (5, 16, 4), (20, 1, 4), (3, 7, 1), (6, 4, 4)])
def test_pages_of_first_tokens_stay(window, keep, page):
    """Whatever the cut, the window's pages and those of the first tokens are there, and no others."""
    rng = random.Random(window * 100 + keep)
    m = CacheManager([PagedNeed(1, 4, window, keep_first=keep)], [None], page, 400, 2, allocate=False)
    for turn in range(2):                                     # the second time on pages used before
        rc = m.add("a")
        done = 0
        while done < 120:
            n = min(rng.choice([1, 1, 2, 5, 17, 40]), 120 - done)
            assert m.reserve("a", done + n)
            first = max(0, done - window + 1)                 # the first key this step's window sees
            need = set(range(first // page, -(-(done + n) // page))) | \
                set(range(-(-min(keep, done + n) // page)))
            assert all(rc.tables[0][p] >= 0 for p in need)
            done += n
            m.advance("a", done)
            m.check()
            first = max(0, done - window + 1)
            for p in range(first // page):
                assert (rc.tables[0][p] >= 0) == (p < -(-keep // page))
        m.free("a")
        assert m.groups[0].pool.in_use == 0


# ---- the plain implementation's mechanisms, each against a form written another way -----------

def test_plain_masks():
    see = plain.visible(50, {"size": 8, "keep_first": 3})
    assert see == [0, 1, 2] + list(range(43, 51))
    assert plain.visible(5, {"size": 8, "keep_first": 3}) == list(range(6))
    assert plain.visible(9, {"size": 8, "keep_first": 3}) == [0, 1, 2] + list(range(2, 10))[1:]
    assert plain.visible(30, {"size": 8}) == list(range(23, 31))
    assert plain.visible(3, None) == [0, 1, 2, 3]


def test_plain_rotations_keep_lengths_and_differences():
    rng = np.random.default_rng(0)
    x, y = rng.standard_normal((2, 16))
    rot = {"dims": 16, "base": 100.0}
    for turn in (plain.rotate_halves, plain.rotate_pairs):
        assert np.allclose(np.linalg.norm(turn(x, 7, rot)), np.linalg.norm(x))
        assert np.allclose(turn(x, 9, rot) @ turn(y, 4, rot), turn(x, 25, rot) @ turn(y, 20, rot))
        part = turn(x, 7, {"dims": 6, "base": 100.0})
        assert np.allclose(part[6:], x[6:]) and not np.allclose(part[:6], x[:6])
    # the two layouts are the same rotation of reordered dimensions
    order = np.concatenate([np.arange(0, 16, 2), np.arange(1, 16, 2)])
    assert np.allclose(plain.rotate_pairs(x, 5, rot)[order], plain.rotate_halves(x[order], 5, rot))
    scaled = {"dims": 16, "base": 100.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    grow = 0.1 * math.log(4.0) + 1.0
    assert np.allclose(np.linalg.norm(plain.rotate_pairs(x, 7, scaled)), grow * np.linalg.norm(x))


def test_position_encodings_have_the_plain_frequencies():
    from rvllm_b200.parts import PositionSpec
    from rvllm_b200.parts.position import PairRope, PartialRope
    for kind, cls in (("rope_partial", PartialRope), ("rope_pairs", PairRope)):
        for dims, base, sc in ((16, 500.0, (4.0, 64, 8.0, 1.0)), (48, 1e5, (2.5, 777, 32.0, 1.5)),
                               (2, 50.0, (8.0, 32, 4.0, 0.5)), (24, 1e4, None), (32, 50.0, (16.0, 4096, 1.0, 0.9))):
            f, m = plain.frequencies(dv._rot(dims, base, sc))
            pe = cls(PositionSpec(kind, head_dim=dims, theta=base, rot_dims=dims, yarn=sc), "cpu")
            inv, n = pe.frequencies()
            assert n == dims and np.allclose(inv.double().numpy(), f, rtol=1e-7)
            assert abs(pe.amplitude - m) < 1e-12


def test_plain_delta_rule_and_state_space_by_sums():
    rng = np.random.default_rng(1)
    T, H, d, n = 9, 2, 3, 4
    # without corrections (beta v only) the delta rule is a sum over tokens when keys are orthogonal
    k = np.zeros((3, 1, 3)); k[range(3), 0, range(3)] = 1.0
    q, v = rng.standard_normal((3, 1, 3)), rng.standard_normal((3, 1, n))
    g, beta = rng.uniform(0.2, 1, (3, 1)), rng.uniform(0.2, 1, (3, 1))
    o, S = plain.delta_rule(q, k, v, g, beta)
    for i in range(3):
        want = sum(q[i, 0, j] * beta[j, 0] * v[j, 0] * np.prod(g[j + 1:i + 1, 0]) for j in range(i + 1))
        assert np.allclose(o[i, 0], want)
    # a token written twice with beta = 1 and no decay is stored once
    one = np.ones((2, 1))
    kk, vv = np.repeat(k[:1], 2, 0), np.repeat(v[:1], 2, 0)
    o, S = plain.delta_rule(kk, kk, vv, one, one)
    assert np.allclose(o[1, 0], v[0, 0]) and np.allclose(S[0], np.outer(k[0, 0], v[0, 0]))
    x, B, C = rng.standard_normal((T, H, n)), rng.standard_normal((T, H, d)), rng.standard_normal((T, H, d))
    dt, a, D = rng.uniform(0.1, 1, (T, H)), rng.uniform(0.2, 1, (T, H)), rng.standard_normal(H)
    y, S = plain.ssd_scan(x, B, C, dt, a, D)
    for i in range(T):
        for h in range(H):
            want = D[h] * x[i, h] + sum(np.prod(a[j + 1:i + 1, h]) * dt[j, h] * (C[i, h] @ B[j, h]) * x[j, h]
                                        for j in range(i + 1))
            assert np.allclose(y[i, h], want)
    y1, s1 = plain.ssd_scan(x[:4], B[:4], C[:4], dt[:4], a[:4], D)
    y2, s2 = plain.ssd_scan(x[4:], B[4:], C[4:], dt[4:], a[4:], D, s1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(s2, S)


def test_plain_convolution_and_grouped_norm():
    x = np.arange(1.0, 9.0).reshape(4, 2)
    f = np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 2.0]])
    got = plain.causal_conv(x, f, np.array([0.5, -1.0]))
    assert np.allclose(got[:, 0], [100.5, 310.5, 531.5, 753.5]) and np.allclose(got[:, 1], 2 * x[:, 1] - 1)
    y = np.array([[3.0, 4.0, 0.0, 2.0]])
    assert np.allclose(plain.grouped_rms(y, 2, 0.0), [[3 / 12.5 ** .5, 4 / 12.5 ** .5, 0.0, 2 / 2 ** .5]])


def test_plain_choice_by_groups():
    s = [0.1, -0.5, -0.2, -0.3, 0.05, -9.0]
    assert plain.choose(s, 3) == [0, 4, 2]
    # groups of two: best scores 0.1, -0.2, 0.05; the two best groups are 0 and 2, so the third choice
    # is a low score of a kept group, not the higher one of the group left out
    assert plain.choose(s, 3, 3, 2) == [0, 4, 1]
    assert plain.choose([-1.0, -2.0, -3.0, -1.5], 2, 2, 1) == [0, 1]       # all negative


# ---- the engine's host side -----------------------------------------------------------------------

@pytest.mark.parametrize("name", ["A", "B", "C"])
@pytest.mark.parametrize("schedule", ["whole", "tail_decode", "portions", "mixed"])
def test_engine_host_side_under_every_cut(folders, name, schedule):
    model, _ = load_model(folders[name], "float32", "cpu", PlainOps())
    vocab = dv.config(name)["vocab"]
    rng = random.Random(5)
    reqs = {f"q{i}": [rng.randrange(vocab) for _ in range(n)]
            for i, n in enumerate((61, 2, 35, 1, 75, 17))}
    steps = schedules.tail_decode(reqs, 12) if schedule == "tail_decode" else \
        getattr(schedules, schedule)(reqs)
    page = 4
    cache = make_cache(model, page, schedules.tokens_held(steps, 64) // page, 4)
    runner = ModelRunner(model, cache, PlainOps())
    got = schedules.replay(runner, steps)
    tensors = dv.read_tensors(folders[name])
    for rid, ids in reqs.items():
        ref = dv.plain_logits(folders[name], name, ids, tensors=tensors).to(torch.float32)
        scale = float(ref.abs().max())
        for p in range(len(ids)):
            assert float((got[(rid, p)] - ref[p]).abs().max()) < 2e-5 * scale, (rid, p)
    assert not cache.requests and all(g.pool.in_use == 0 for g in cache.groups)


def test_parts_refuse_what_they_cannot_do():
    from rvllm_b200.parts import AttentionSpec, GatedDeltaSpec, MoESpec, StateSpaceSpec, mixer_class
    from rvllm_b200.parts.feed_forward import MoE
    for spec in (AttentionSpec("attention", 8, num_heads=2, num_kv_heads=1, head_dim=4, keep_first=3),
                 GatedDeltaSpec("gated_delta", 8, num_heads=2, num_kv_heads=1, head_dim=4, v_head_dim=4,
                                taps=2, decay="head", decay_rank=2),
                 GatedDeltaSpec("gated_delta", 8, num_heads=2, num_kv_heads=1, head_dim=4, v_head_dim=4,
                                taps=2, decay="channel"),
                 StateSpaceSpec("state_space", 8, num_heads=3, v_head_dim=4, state=4, groups=2, taps=2)):
        with pytest.raises(ValueError):
            mixer_class(spec.kind).params(spec)
    with pytest.raises(ValueError):
        MoE.params(MoESpec("moe", 8, ffn_dim=4, experts=3, identity=2, top=6))
