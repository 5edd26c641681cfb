"""Fekizen without a GPU: its configuration, its tensor declarations, the plain implementation's
own mechanisms, and the engine's host side (a window's pages beside the rows of pooled blocks, a
state record beside a mixer's own cache, batch packing, step function) driven through the plain
kernel references against the plain implementation of the whole design."""
import math
import random

import numpy as np
import pytest
import torch

import fekizen_tiny as fk
import plain_fekizen as plain
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
    root = str(tmp_path_factory.mktemp("fk"))
    return {n: fk.write(root, n) for n in fk.CONFIGS}


def test_config_round_trip_and_errors():
    for name in fk.CONFIGS:
        cfg = config_from_dict(fk.config(name))
        assert config_from_dict(cfg.to_dict()) == cfg
        assert cfg.architecture == "Fekizen"

    def refused(change):
        bad = fk.config("A")
        change(bad)
        with pytest.raises(ConfigError):
            config_from_dict(bad)

    left = lambda c: c["layers"][1]["mixer"]["left"]
    refused(lambda c: left(c).update(kv_heads=4))                  # does not divide the heads
    refused(lambda c: left(c).update(vdim=16))                     # the values are the keys
    refused(lambda c: left(c)["rot"].update(dims=34))              # more than a head has
    refused(lambda c: left(c)["mask"].update(size=0))
    refused(lambda c: c["layers"][0]["mixer"].update(decay=[0.5])) # one number per head
    refused(lambda c: c["loop"].update(stop=5))                    # beyond the last layer
    refused(lambda c: c["layers"][0]["mlp"]["router"].update(top=7))
    refused(lambda c: c["layers"][0].update(type="sideways"))
    refused(lambda c: c["layers"][1]["mixer"].pop("right"))
    refused(lambda c: c["layers"][1]["mixer"]["right"].update(tau=0))
    refused(lambda c: c.pop("max_positions"))


def test_rank_comes_from_the_tensor_file():
    data = fk.config("A")
    for i in (1, 3):
        del data["layers"][i]["mixer"]["right"]["rank"]
    cfg = config_from_dict(data)
    with pytest.raises(ConfigError):
        cfg.with_tensor_shapes({})
    full = cfg.with_tensor_shapes({"l1.mix.right.a1": (8, 96), "l3.mix.right.a1": (12, 96)})
    assert full == config_from_dict(fk.config("A"))
    with pytest.raises(ConfigError):
        full.with_tensor_shapes({"l1.mix.right.a1": (9, 96), "l3.mix.right.a1": (12, 96)})


def test_declared_tensors_and_run_order():
    cfg = config_from_dict(fk.config("A"))
    spec = architecture("Fekizen").build_spec(cfg)
    decls = param_decls(spec)
    shapes = {n: d.shape for n, d in decls.items()}
    assert shapes["embed"] == (300, 96) and shapes["pos"] == (512, 96)
    assert shapes["loop.step"] == (3, 96) and shapes["l2.shift"] == (96,)
    assert shapes["l0.mix.q"] == (48, 96) and shapes["l0.mix.norm"] == (72,)
    assert shapes["l1.mix.left.q"] == (192, 96) and shapes["l1.mix.left.k"] == (64, 96)
    assert "l1.mix.left.v" not in shapes and shapes["l1.mix.left.sink"] == (6,)
    assert shapes["l1.mix.left.out"] == shapes["l1.mix.right.out"] == (96,)
    assert shapes["l1.mix.right.a1"] == (8, 96) and shapes["l1.mix.right.a2"] == (48, 8)
    assert shapes["l1.mix.right.a2.b"] == (48,) and shapes["l1.mix.right.norm"] == (16,)
    assert shapes["l0.mlp.e5.gate"] == (32, 96) and shapes["l0.mlp.shared.down"] == (96, 48)
    assert "l1.mlp.shared.up" not in shapes and "l2.norm2" not in shapes
    # layer 0, then layers 1 and 2 three times, then layer 3; from the second pass on the rows the
    # first layer read are added once more
    assert [(c.layer, c.add, c.add_start) for c in spec.order] == [
        (0, None, False), (1, ("loop.step", 0), False), (2, None, False),
        (1, ("loop.step", 1), True), (2, None, False), (1, ("loop.step", 2), True),
        (2, None, False), (3, None, False)]
    spec_b = architecture("Fekizen").build_spec(config_from_dict(fk.config("B")))
    assert [c.layer for c in spec_b.order] == [0, 1, 2] and "loop.step" not in param_decls(spec_b)


def test_what_a_call_remembers(folders):
    model, _ = load_model(folders["A"], "float32", "cpu", PlainOps())
    needs = model.cache_needs()
    assert needs[0] == SeveralNeeds((StateNeed((3 * 16 * 24,)), StateNeed((96,))))
    window = SeveralNeeds((PagedNeed(2, 32, 20, block=8), PagedNeed(2, 32, every=8)))
    assert needs[1] == needs[3] == needs[5] == SeveralNeeds(
        (SeveralNeeds((window, StateNeed((2 * 24 * 16,)))), StateNeed((96,))))
    cache = make_cache(model, 4, 32, 2)
    mixer, last = cache.views()[1].parts
    (tokens, blocks), memory = mixer.parts[0].parts, mixer.parts[1]
    assert (tokens.kind, blocks.kind, memory.kind, last.kind) == ("paged", "paged", "state", "state")
    assert tokens.group != blocks.group
    # every pass writes pages and records of its own
    other = cache.views()[3].parts[0].parts[0].parts
    assert other[0].k.data_ptr() != tokens.k.data_ptr()
    assert other[1].k.data_ptr() != blocks.k.data_ptr()


# ---- the cache: one row per block -----------------------------------------------------------

def _pooled_manager(window, pool, page, pages, slots=3):
    need = SeveralNeeds((PagedNeed(1, 4, window, block=pool), PagedNeed(1, 4, every=pool)))
    return CacheManager([need], [None], page, pages, slots, allocate=False)


def test_rows_of_blocks_take_a_page_per_page_of_blocks():
    m = _pooled_manager(window=8, pool=4, page=2, pages=40)
    assert m.groups[1].pool.num_pages == 10 + 3
    rc = m.add("a")
    assert m.pages_needed("a", 3) == [2, 0]                  # no block is complete
    assert m.pages_needed("a", 4) == [2, 1] and m.pages_needed("a", 11) == [6, 1]
    assert m.pages_needed("a", 12) == [6, 2]                 # three blocks, two rows a page
    assert m.reserve("a", 12) and [len(t) for t in rc.tables] == [6, 2]
    m.check()
    m.free("a")
    assert all(g.pool.in_use == 0 for g in m.groups)


@pytest.mark.parametrize("window,pool,page", [(8, 4, 2), (5, 7, 2), (3, 16, 4), (20, 3, 4), (1, 1, 1)])
def test_pages_stay_until_window_and_block_have_passed(window, pool, page):
    """Whatever the cut, the pages of every token that a later step reads are there: the window's,
    and those of the block that is not complete yet."""
    rng = random.Random(window * 100 + pool)
    m = _pooled_manager(window, pool, page, 400)
    rc = m.add("a")
    done = 0
    while done < 150:
        n = min(rng.choice([1, 1, 2, 5, 17, 40]), 150 - done)
        assert m.reserve("a", done + n)
        first = min(max(0, done - window + 1), done // pool * pool)   # what this step reads
        assert all(p >= 0 for p in rc.tables[0][first // page:])
        assert all(p >= 0 for p in rc.tables[1])
        done += n
        m.advance("a", done)
        m.check()
        first = min(max(0, done - window + 1), done // pool * pool)
        assert all(p < 0 for p in rc.tables[0][:first // page])       # and no others
    m.free("a")


def test_room_counts_rows_of_blocks():
    m = _pooled_manager(window=8, pool=4, page=2, pages=10)
    assert m.room() == 20                                     # ten pages of two tokens
    m.add("a")
    m.reserve("a", 7)
    assert m.room("a") == 20 and m.room() == 12
    while m.groups[1].pool.available:                         # no row of a block left
        m.groups[1].pool.alloc()
    # a's one page of rows holds two blocks: 11 tokens complete no third one
    assert m.room("a") == 11 and m.room() == 3


# ---- the plain implementation's mechanisms, each against a form written another way -----------

def test_plain_yarn_frequencies():
    rot = {"dims": 8, "base": 100.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    f, m = plain.yarn_frequencies(rot)
    plainf = np.array([100.0 ** (-2 * i / 8) for i in range(4)])
    # dim(8) = 8 ln(64 / 16 pi) / (2 ln 100) = 0.21 -> lo 0; dim(1) = 2.02 -> hi 3
    ramp = np.array([0.0, 1 / 3, 2 / 3, 1.0])
    assert np.allclose(f, plainf * (1 - ramp) + plainf / 4.0 * ramp)
    assert abs(m - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    f, m = plain.yarn_frequencies({"dims": 8, "base": 100.0})
    assert np.allclose(f, plainf) and m == 1.0
    # one turn over the whole context is exactly the last dimension at most: a clamp at dims - 1
    rot["scaling"]["slow"] = 1e-9
    f, _ = plain.yarn_frequencies(rot)
    assert np.allclose(f, plainf * (1 - np.arange(4) / 7) + plainf / 4.0 * (np.arange(4) / 7))


def test_position_encoding_has_the_plain_frequencies():
    from rvllm_b200.parts import PositionSpec
    from rvllm_b200.parts.position import PartialRope
    for dims, head, base, sc in ((16, 32, 500.0, (4.0, 64, 8.0, 1.0)), (48, 48, 1e5, (2.5, 777, 32.0, 1.5)),
                                 (6, 10, 2e5, (8.0, 32, 4.0, 0.5)), (24, 24, 1e4, None),
                                 (32, 32, 50.0, (16.0, 4096, 1.0, 0.9))):
        rot = fk._rot(dims, base, sc)
        f, m = plain.yarn_frequencies(rot)
        pe = PartialRope(PositionSpec("rope_partial", head_dim=head, theta=base, rot_dims=dims,
                                      yarn=sc), "cpu")
        inv, n = pe.frequencies()
        assert n == dims and np.allclose(inv.double().numpy(), f, rtol=1e-7)
        assert abs(pe.amplitude - m) < 1e-12


def test_plain_seen_blocks_at_every_edge():
    for size, pool in ((8, 4), (5, 7), (3, 16), (1, 1), (13, 13), (20, 3)):
        for i in range(120):
            nb = plain.seen_blocks(i, size, pool)
            assert nb == max(0, i - size + 1) // pool
            assert nb == 0 or nb * pool - 1 <= i - size            # the last block is wholly before
            assert (nb + 1) * pool - 1 > i - size                  # the next one is not


def test_plain_recurrence_equals_its_unrolled_sum():
    rng = np.random.default_rng(1)
    T, H, d, dv = 9, 2, 3, 4
    q, k = rng.standard_normal((T, H, d)), rng.standard_normal((T, H, d))
    v, a = rng.standard_normal((T, H, dv)), rng.uniform(0.2, 1.0, (T, H, d))
    got, S = plain.recurrence(q, k, v, a)
    for i in range(T):
        for h in range(H):
            want = sum(((q[i, h] * np.prod(a[j + 1:i + 1, h], axis=0)) @ k[j, h]) * v[j, h]
                       for j in range(i + 1))
            assert np.allclose(got[i, h], want)
    o1, s1 = plain.recurrence(q[:4], k[:4], v[:4], a[:4])
    o2, s2 = plain.recurrence(q[4:], k[4:], v[4:], a[4:], s1)
    assert np.allclose(np.concatenate([o1, o2]), got) and np.allclose(s2, S)


def test_plain_attend_counts_the_sink_once_and_caps_scores():
    q = np.array([2.0, 0.0])
    keys, vals = np.array([[30.0, 0.0], [1.0, 5.0]]), np.array([[1.0, 0.0], [0.0, 1.0]])
    s = 4.0 * np.tanh(np.array([30.0, 1.0]) * 2.0 * 0.5 / 4.0)
    den = np.exp(s).sum() + math.exp(1.5)
    assert np.allclose(plain.attend(q, keys, vals, 0.5, 4.0, 1.5), np.exp(s) / den)
    s = np.array([30.0, 1.0])
    den = np.exp(s).sum() + math.exp(100.0)
    assert np.allclose(plain.attend(q, keys, vals, 0.5, None, 100.0), np.exp(s) / den)


def test_plain_token_shift_and_route():
    h = np.arange(6.0).reshape(3, 2) + 1.0
    mix = np.array([0.25, 1.0])
    assert np.allclose(plain.token_shift(h, mix), [[0.75, 0.0], [2.5, 2.0], [4.5, 4.0]])
    chosen, w = plain.route(np.array([0.1, 3.0, -2.0, 2.0]), 2)
    assert list(chosen) == [1, 3] and np.allclose(w, np.exp([0.0, -1.0]) / np.exp([0.0, -1.0]).sum())


# ---- the engine's host side -----------------------------------------------------------------------

@pytest.mark.parametrize("name", ["A", "B", "C"])
@pytest.mark.parametrize("schedule", ["whole", "tail_decode", "portions", "mixed"])
def test_engine_host_side_under_every_cut(folders, name, schedule):
    model, _ = load_model(folders[name], "float32", "cpu", PlainOps())
    vocab = fk.config(name)["vocab"]
    rng = random.Random(5)
    reqs = {f"q{i}": [rng.randrange(vocab) for _ in range(n)]
            for i, n in enumerate((61, 2, 35, 1, 75, 17))}
    steps = schedules.tail_decode(reqs, 12) if schedule == "tail_decode" else \
        getattr(schedules, schedule)(reqs)
    page = 4
    cache = make_cache(model, page, schedules.tokens_held(steps, 64) // page, 4)
    runner = ModelRunner(model, cache, PlainOps())
    got = schedules.replay(runner, steps)
    tensors = fk.read_tensors(folders[name])
    for rid, ids in reqs.items():
        ref = fk.plain_logits(folders[name], name, ids, tensors=tensors).to(torch.float32)
        scale = float(ref.abs().max())
        for p in range(len(ids)):
            assert float((got[(rid, p)] - ref[p]).abs().max()) < 2e-5 * scale, (rid, p)
    assert not cache.requests and all(g.pool.in_use == 0 for g in cache.groups)


def test_the_context_ends_with_the_position_table(folders):
    model, _ = load_model(folders["C"], "float32", "cpu", PlainOps())
    runner = ModelRunner(model, make_cache(model, 16, 40, 1), PlainOps())
    runner.add_request("a")
    from rvllm_b200.engine import StepEntry
    with pytest.raises(ValueError):
        runner.step([StepEntry("a", [1] * 451, ())])
