"""Fekizen on the GPU against the plain implementation (tests/plain_fekizen.py): each new kernel
alone at sizes other than any model's, with inputs made so that a fault shows; models of one
mechanism each, with attention made sharp so that one lost key changes the result; then the
engine under every way of cutting requests into steps, in float32 and bfloat16, with and without
replayed launch sequences; then greedy generation through the Python entry point and its
scheduler, and the programs a user starts."""
import copy
import os
import random
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import fekizen_tiny as fk
import plain_fekizen as plain
import schedules

pytestmark = pytest.mark.gpu
BOUND = {"float32": 2e-5, "bfloat16": 3e-2}


@pytest.fixture(scope="module")
def ops():
    from rvllm_b200.kernels import cuda_ops
    return cuda_ops()


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = str(tmp_path_factory.mktemp("fk"))
    return {n: fk.write(root, n) for n in fk.CONFIGS}


def dev(t, dtype=None):
    return t.to("cuda", dtype) if dtype is not None else t.to("cuda")


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def close(got, want, dtype, scale=None, bound=None):
    want = torch.as_tensor(np.asarray(want), dtype=torch.float64)
    got = got.detach().to("cpu", torch.float64).reshape(want.shape)
    s = float(want.abs().max()) if scale is None else scale
    err = float((got - want).abs().max()) / max(s, 1e-30)
    assert err < max(bound or 0.0, 1e-5 if dtype == torch.float32 else 2e-2), err


def rnd(gen, dtype, *shape, std=1.0):
    """Random values that both sides can hold exactly."""
    return (torch.randn(*shape, generator=gen) * std).to(dtype).double()


def step_context(layout):
    """Index arrays of a step: `layout` lists (tokens, state slot) per request."""
    starts, token_req = [0], []
    for r, (n, _) in enumerate(layout):
        starts.append(starts[-1] + n)
        token_req += [r] * n
    n_decode = 0
    while n_decode < len(layout) and layout[n_decode][0] == 1:
        n_decode += 1
    return SimpleNamespace(q_start=i32(starts), state_slot=i32([s for _, s in layout]),
                           token_req=i32(token_req), n_reqs=len(layout), n_decode=n_decode,
                           n_tokens=starts[-1]), starts


# ---- embedding rows with positions ---------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [64, 50])
def test_embedding_adds_unscaled_positions(ops, dtype, width):
    g = torch.Generator().manual_seed(width)
    table, pos = rnd(g, dtype, 31, width), rnd(g, dtype, 20, width)
    ids, where = [3, 30, 0, 3, 7], [0, 19, 4, 4, 1]
    out = torch.empty(5, width, device="cuda")
    ops.embed(dev(table, dtype), i32(ids), out, 2.5, positions=i32(where), position_table=dev(pos, dtype))
    close(out, 2.5 * table[ids] + pos[where], torch.float32)


# ---- norm with a token shift ------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [96, 50, 1024, 2600])
@pytest.mark.parametrize("big", [False, True])
def test_norm_moves_rows_towards_the_token_before(ops, dtype, width, big):
    """Requests of one, two and many tokens, a filling request without a slot, records that are
    not in order; with few rows (a row a block) and many (several)."""
    g = torch.Generator().manual_seed(width)
    layout = [(1, 4), (1, -1), (1, 0), (9, 2), (2, 5), (0, -1), (330 if big else 6, 1), (3, -1)]
    ctx, starts = step_context(layout)
    n, eps = ctx.n_tokens, 1e-4
    resid, delta = rnd(g, torch.float32, n, width), rnd(g, dtype, n, width)
    extra, add = rnd(g, torch.float32, n, width), rnd(g, torch.float32, width)
    scale, mix = rnd(g, torch.float32, width), rnd(g, torch.float32, width)
    weight, state = rnd(g, torch.float32, width), rnd(g, torch.float32, 6, width)
    for use in ((1, 1, 1, 1), (1, 0, 0, 0), (0, 0, 1, 1), (0, 0, 0, 0)):
        x = resid.clone()
        x = x + (delta * scale if use[1] else delta) if use[0] else x
        x = x + extra if use[2] else x
        x = x + add if use[3] else x
        h = torch.as_tensor(plain.rms(x.numpy(), eps)) * weight
        want, rec = h.clone(), state.clone()
        for (m, slot), a in zip(layout, starts):
            for t in range(a, a + m):
                before = h[t - 1] if t > a else (state[slot] if slot >= 0 else torch.zeros_like(h[t]))
                want[t] = h[t] + (before - h[t]) * mix
            if m and slot >= 0:
                rec[slot] = h[a + m - 1]
        r, st = dev(resid.float()), dev(state.float())
        new, out = torch.empty_like(r), torch.empty(n, width, device="cuda", dtype=dtype)
        opt = dict(delta_scale=dev(scale.float()) if use[1] else None,
                   add_rows=dev(extra.float()) if use[2] else None,
                   add=dev(add.float()) if use[3] else None)
        d = dev(delta, dtype) if use[0] else None
        ops.add_rmsnorm_shift(r, new, d, dev(weight.float()), eps, out, ctx, dev(mix.float()), st, **opt)
        close(out, want, dtype)
        close(new, x, torch.float32)
        close(st, rec, torch.float32)
        close(r, resid, torch.float32)                       # the rows it was given stay
        # without a shift the stream is updated in place
        ops.add_rmsnorm_shift(r, r, d, dev(weight.float()), eps, out, ctx, None, None, **opt)
        close(out, h, dtype)
        close(r, x, torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sum_of_two_normed_branches(ops, dtype):
    g = torch.Generator().manual_seed(3)
    for n, w in ((5, 48), (33, 50), (40, 1024), (2, 3000)):
        a, b = rnd(g, dtype, n, w, std=3.0), rnd(g, dtype, n, w, std=0.01)
        wa, wb = rnd(g, torch.float32, w), rnd(g, torch.float32, w)
        out = torch.empty(n, w, device="cuda", dtype=dtype)
        ops.normed_sum(dev(a, dtype), dev(wa.float()), 0.5, dev(b, dtype), dev(wb.float()), 0.7, 1e-5, out)
        close(out, 0.5 * plain.rms(a.numpy(), 1e-5) * wa.numpy() + 0.7 * plain.rms(b.numpy(), 1e-5) * wb.numpy(), dtype)


# ---- rotation, values that are keys, the rows of pooled blocks ------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(6, 2, 32, 16), (3, 3, 10, 6), (4, 1, 48, 48), (2, 2, 16, 0)])
def test_rotation_with_amplitude_and_values_that_are_keys(ops, dtype, sizes):
    H, G, d, dims = sizes
    g = torch.Generator().manual_seed(d)
    rot = fk._rot(dims, 300.0, (4.0, 64, 8.0, 1.0)) if dims else None
    positions = [0, 1, 2, 17, 333, 5, 90]
    n = len(positions)
    rows = rnd(g, dtype, n, (H + G) * d)
    slots = [3, 9, 0, -1, 14, 7, 1]
    freq = None
    amp = 1.0
    if dims:
        f, amp = plain.yarn_frequencies(rot)
        freq = (dev(torch.from_numpy(f).float()), dims)
    k = torch.full((4, 4, G, d), 9.0, device="cuda", dtype=dtype)
    v = torch.full((4, 4, G, d), 9.0, device="cuda", dtype=dtype)
    x = dev(rows, dtype)
    ops.rope_partial_write(x, H, G, d, d, freq, i32(positions), i32(slots), k, v, amplitude=amp,
                           values_are_keys=True)
    q, kk = rows[:, :H * d].reshape(n, H, d).numpy(), rows[:, H * d:].reshape(n, G, d).numpy()
    close(x[:, :H * d], np.stack([plain.rotate(q[t], positions[t], rot) for t in range(n)]), dtype, bound=5e-5)
    kp, vp = k.reshape(16, G, d), v.reshape(16, G, d)
    for t, s in enumerate(slots):
        if s >= 0:
            close(kp[s], plain.rotate(kk[t], positions[t], rot), dtype, bound=5e-5)
            close(vp[s], kk[t], dtype)                       # as projected, before the rotation
    untouched = [s for s in range(16) if s not in slots]
    assert float((kp[untouched] - 9.0).abs().max()) == 0 and float((vp[untouched] - 9.0).abs().max()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(6, 3, 10, 6, 7), (8, 2, 64, 64, 16), (5, 5, 16, 0, 1), (4, 1, 80, 16, 40)])
@pytest.mark.parametrize("v_is_k", [True, False])
def test_rows_of_blocks_are_means_of_the_cached_rows(ops, dtype, sizes, v_is_k):
    """Three requests in portions of every kind against pool borders: queries, cached rows and the
    blocks' rows, which are the means of the rows as they are cached, whatever the cut."""
    H, G, d, dims, pool = sizes
    page, n_req = 4, 3
    lengths = (95, 41, pool)
    rot = fk._rot(dims, 300.0, (4.0, 64, 8.0, 1.0)) if dims else None
    freq, amp = None, 1.0
    if dims:
        f, amp = plain.yarn_frequencies(rot)
        freq = (dev(torch.from_numpy(f).float()), dims)
    g = torch.Generator().manual_seed(d)
    rows = [rnd(g, dtype, n, (H + G * (1 if v_is_k else 2)) * d) for n in lengths]
    rng = random.Random(pool)
    ids = rng.sample(range(60), 60)
    table = torch.tensor([ids[20 * r:20 * r + 24] if r < 2 else ids[40:60] + [-1] * 4 for r in range(3)],
                         dtype=torch.int32)
    table[0] = torch.tensor(ids[:24]); table[1] = torch.tensor(ids[24:48]); table[2, :12] = torch.tensor(ids[48:60])
    pids = rng.sample(range(140), 140)                       # rows of blocks, anywhere
    k = torch.full((60, page, G, d), 9.0, device="cuda", dtype=dtype)
    v = torch.full_like(k, 9.0)
    kb = torch.full((35, 4, G, d), 9.0, device="cuda", dtype=dtype)
    vb = torch.full_like(kb, 9.0)
    done = [0, 0, 0]
    cuts = [[1, 1, 39, 2, 3, 49], [2, 30, 1, 1, 7], [pool]]
    qs = [[], [], []]
    for step in range(6):
        parts = [(r, cuts[r][step]) for r in range(n_req) if step < len(cuts[r])]
        parts.sort(key=lambda x: x[1] != 1)
        layout = [(m, 0) for _, m in parts] + [(3, -1)]      # a filling request writes nothing
        ctx, starts = step_context(layout)
        pos, slots, done_slots, x = [], [], [], []
        for r, m in parts:
            for p in range(done[r], done[r] + m):
                pos.append(p)
                slots.append(int(table[r, p // page]) * page + p % page)
                done_slots.append(pids[r * 45 + p // pool] if (p + 1) % pool == 0 and p // pool < 45 else -1)
            x.append(rows[r][done[r]:done[r] + m])
        ctx.positions = i32(pos + [0] * 3)
        tabs = torch.cat([table[[r for r, _ in parts]], torch.full((1, 24), -1, dtype=torch.int32)])
        group = SimpleNamespace(block_table=dev(tabs), max_blocks=24, page_size=page,
                                slot_mapping=i32(slots + [-1] * 3))
        xs = dev(torch.cat(x + [torch.full((3, rows[0].shape[1]), 50.0, dtype=torch.float64)]), dtype)
        ops.rope_pool_write(xs, H, G, d, freq, ctx, group, k, v, pool, i32(done_slots + [-1] * 3), kb, vb,
                            amplitude=amp, values_are_keys=v_is_k)
        for (r, m), a in zip(parts, starts):
            qs[r].append(xs[a:a + m, :H * d].cpu())
            done[r] += m
    written, wrows = set(), set()
    for r, n in enumerate(lengths[:2] + (pool,)):
        n = done[r]
        q = rows[r][:n, :H * d].reshape(n, H, d).numpy()
        kk = rows[r][:n, H * d:(H + G) * d].reshape(n, G, d).numpy()
        vv = kk if v_is_k else rows[r][:n, (H + G) * d:].reshape(n, G, d).numpy()
        close(torch.cat(qs[r]), np.stack([plain.rotate(q[t], t, rot) for t in range(n)]), dtype, bound=5e-5)
        at = [int(table[r, p // page]) * page + p % page for p in range(n)]
        written |= set(at)
        ck, cv = k.reshape(-1, G, d)[at].cpu().double(), v.reshape(-1, G, d)[at].cpu().double()
        close(ck, np.stack([plain.rotate(kk[t], t, rot) for t in range(n)]), dtype, bound=5e-5)
        assert float((cv - torch.from_numpy(vv)).abs().max()) == 0
        for b in range(min(n // pool, 45)):
            s = pids[r * 45 + b]
            wrows.add(s)
            close(kb.reshape(-1, G, d)[s], ck[b * pool:(b + 1) * pool].mean(0), dtype, scale=1.0)
            close(vb.reshape(-1, G, d)[s], cv[b * pool:(b + 1) * pool].mean(0), dtype, scale=1.0)
    for t, used in ((k, written), (v, written), (kb, wrows), (vb, wrows)):
        rest = [s for s in range(t.shape[0] * t.shape[1]) if s not in used]
        assert float((t.reshape(-1, G, d)[rest] - 9.0).abs().max()) == 0


# ---- attention over a window and the blocks before it ------------------------------------------------------

class _Pages:
    """Keys and values of requests scattered over pages in random order, with their blocks' rows."""

    def __init__(self, gen, dtype, lengths, G, d, page, pool, window):
        rng = random.Random(d + page)
        self.k = [rnd(gen, dtype, n, G, d) for n in lengths]
        self.v = [rnd(gen, dtype, n, G, d) for n in lengths]
        self.pool, self.page, self.dtype, self.lengths, self.window = pool, page, dtype, lengths, window
        blocks = [-(-n // page) for n in lengths]
        ids = rng.sample(range(sum(blocks) + 3), sum(blocks))
        pblocks = [-(-(n // pool) // page) if pool else 0 for n in lengths]
        pids = rng.sample(range(sum(pblocks) + 3), sum(pblocks))
        self.table = torch.full((len(lengths), max(blocks) + 1), -1, dtype=torch.int32)
        self.ptable = torch.full((len(lengths), max(pblocks) + 1), -1, dtype=torch.int32)
        a = b = 0
        for r in range(len(lengths)):
            self.table[r, :blocks[r]] = torch.tensor(ids[a:a + blocks[r]], dtype=torch.int32)
            self.ptable[r, :pblocks[r]] = torch.tensor(pids[b:b + pblocks[r]], dtype=torch.int32)
            a, b = a + blocks[r], b + pblocks[r]
        self.shape = (sum(blocks) + 3, page, G, d)
        self.pshape = (sum(pblocks) + 3, page, G, d)

    def rows(self, r):
        """The block rows as the cache holds them (rounded to the storage type)."""
        n, P = self.lengths[r] // self.pool, self.pool
        return [x[r][:n * P].reshape(n, P, *x[r].shape[1:]).mean(1).to(self.dtype).double()
                for x in (self.k, self.v)]

    def build(self, released):
        """Device pages; with `released`, entries of pages wholly before what is read are -1 and
        everything that is not a cached row is large, so that reading it would show."""
        k, v = (torch.full(self.shape, 50.0, dtype=torch.float64) for _ in range(2))
        pk, pv = (torch.full(self.pshape, 50.0, dtype=torch.float64) for _ in range(2))
        table = self.table.clone()
        for r, n in enumerate(self.lengths):
            for j in range(n):
                k[int(self.table[r, j // self.page]), j % self.page] = self.k[r][j]
                v[int(self.table[r, j // self.page]), j % self.page] = self.v[r][j]
            if self.pool:
                kb, vb = self.rows(r)
                for j in range(n // self.pool):
                    at = (int(self.ptable[r, j // self.page]), j % self.page)
                    pk[at], pv[at] = kb[j], vb[j]
            if released is not None and self.window:
                first = max(0, released[r] - self.window + 1) // self.page
                for p in table[r, :first].tolist():
                    k[p], v[p] = 50.0, 50.0
                table[r, :first] = -1
        c = lambda t: dev(t, self.dtype)
        group = SimpleNamespace(block_table=dev(table), max_blocks=table.shape[1], page_size=self.page)
        pooled = None
        if self.pool:
            pg = SimpleNamespace(block_table=dev(self.ptable), max_blocks=self.ptable.shape[1], page_size=self.page)
            pooled = (c(pk), c(pv), pg, self.pool)
        return c(k), c(v), group, pooled


def _attention_case(ops, dtype, sizes, lengths, new, page, pool, window, scale, cap, loud=()):
    """`new[r]`: the last new[r] tokens of request r are this step's.  `loud`: (request, position of
    the key, position of the query): the query is made to point at that key (or at its block's
    mean), so that one score stands out among all."""
    H, G, d = sizes
    g = torch.Generator().manual_seed(H * d + page)
    pages = _Pages(g, dtype, lengths, G, d, page, pool, window)
    q = [rnd(g, dtype, n, H, d) for n in lengths]
    sinks = rnd(g, torch.float32, H)
    for r, kp, qp in loud:
        # eight times the key: its score is far above all others'
        q[r][qp] = (pages.k[r][kp].repeat_interleave(H // G, dim=0) * 8.0).to(dtype).double()
    starts = [n - m for n, m in zip(lengths, new)]
    order = sorted(range(len(lengths)), key=lambda r: new[r] != 1)
    assert order == list(range(len(lengths)))
    k, v, group, pooled = pages.build(starts)
    rows = torch.cat([q[r][starts[r]:].reshape(new[r], H * d) for r in order])
    extra = rnd(g, dtype, rows.shape[0], G * d)              # keys ride behind the queries
    ctx, cum = step_context([(m, 0) for m in new])
    ctx.ctx_lens = i32(lengths)
    ctx.max_q_len, ctx.max_ctx_len = max(new), max(lengths)
    out = torch.full((rows.shape[0], H * d), float("nan"), device="cuda", dtype=dtype)
    ops.paged_attention_pooled(dev(torch.cat([rows, extra], 1).contiguous(), dtype), H, G, d, k, v, ctx, group,
                               pooled, scale, cap, window, dev(sinks.float()), out)
    # a launch made for longer contexts (as replayed steps are) gives the same
    ctx.max_ctx_len = 4 * max(lengths)
    out2 = torch.empty_like(out)
    ops.paged_attention_pooled(dev(torch.cat([rows, extra], 1).contiguous(), dtype), H, G, d, k, v, ctx, group,
                               pooled, scale, cap, window, dev(sinks.float()), out2)
    for r in order:
        kb, vb = pages.rows(r) if pool else (None, None)
        for t in range(new[r]):
            p = starts[r] + t
            lo = max(0, p - window + 1) if window else 0
            nb = plain.seen_blocks(p, window, pool) if pool else 0
            for h in range(H):
                gg = h // (H // G)
                keys, vals = pages.k[r][lo:p + 1, gg], pages.v[r][lo:p + 1, gg]
                if nb:
                    keys, vals = torch.cat([kb[:nb, gg], keys]), torch.cat([vb[:nb, gg], vals])
                want = plain.attend(q[r][p, h].numpy(), keys.numpy(), vals.numpy(), scale, cap, float(sinks[h]))
                for o in (out, out2):
                    close(o[cum[r] + t, h * d:(h + 1) * d], want, dtype, scale=1.0,
                          bound=5e-5 if dtype == torch.float32 else 3e-2)


SHAPES = [(torch.float32, (4, 2, 32)), (torch.float32, (3, 1, 10)), (torch.bfloat16, (8, 2, 64)),
          (torch.bfloat16, (6, 2, 48)), (torch.bfloat16, (3, 3, 10)), (torch.bfloat16, (20, 1, 16)),
          (torch.bfloat16, (2, 1, 128))]


@pytest.mark.parametrize("dtype,sizes", SHAPES)
@pytest.mark.parametrize("window,pool,cap", [(20, 8, 15.0), (13, 13, None), (5, 7, 30.0), (64, 16, 9.0), (None, None, 12.0)])
def test_pooled_attention_every_visible_key(ops, dtype, sizes, window, pool, cap):
    d = sizes[2]
    _attention_case(ops, dtype, sizes, (150, 1, 33, 70, 129), (1, 1, 1, 70, 67), 8, pool, window, d ** -0.5, cap)


@pytest.mark.parametrize("dtype,sizes", [SHAPES[0], SHAPES[2], SHAPES[4]])
@pytest.mark.parametrize("decoded", [True, False])
def test_one_key_stands_out_at_every_edge(ops, dtype, sizes, decoded):
    """For one query the window's oldest key and the one before it, a position hidden between the
    window and the newest mean, the ends of the newest mean's block, of the one after it and of the
    oldest, page borders: each made the one whose score stands out."""
    window, pool, page, n = 40, 8, 16, 200
    P = n - 1                                                # the last query
    nb = plain.seen_blocks(P, window, pool)
    edges = [P, P - 1, P - window + 1, P - window, nb * pool, nb * pool - 1, (nb - 1) * pool, 0, pool - 1,
             page, page - 1, 176, 175]
    for e in edges:
        new = (1,) if decoded else (70,)
        _attention_case(ops, dtype, sizes, (n,), new, page, pool, window, sizes[2] ** -0.5, None,
                        loud=[(0, e, P)])


@pytest.mark.parametrize("dtype,sizes", [SHAPES[0], SHAPES[2]])
def test_many_blocks_and_windows_beyond_a_split(ops, dtype, sizes):
    """More than 256 blocks before the window and windows of more than 256 tokens: single tokens
    are split over both, and a far block among hundreds stands out."""
    for window, pool, lengths in ((30, 3, (1000, 900)), (600, 4, (1900, 700)), (257, 2, (1101, 300))):
        loud = [(0, 5, lengths[0] - 1), (1, lengths[1] - window, lengths[1] - 1)]
        _attention_case(ops, dtype, sizes, lengths, (1, 1), 16, pool, window, 0.2, 40.0, loud=loud)
    _attention_case(ops, dtype, sizes, (1000,), (20,), 16, 3, 30, 0.2, None, loud=[(0, 5, 999), (0, 300, 985)])


# ---- linear attention ----------------------------------------------------------------------------------

def _memory(gen, H, d, dv, constant, silu, head_norm, silu_gate, n):
    m = SimpleNamespace(H=H, d=d, dv=dv, silu=silu, head=head_norm, gate=silu_gate, tau=3.0, eps=1e-5,
                        q_scale=0.7)
    m.rows = rnd(gen, torch.bfloat16, n, 2 * H * d + 2 * H * dv).numpy()     # both types hold these
    m.z = None if constant else rnd(gen, torch.float32, n, H * d).numpy()
    m.log_decay = np.log(np.linspace(0.3, 0.999, H)) if constant else None
    m.bias = None if constant else rnd(gen, torch.float32, H * d).numpy()
    m.norm = 1.0 + 0.1 * rnd(gen, torch.float32, H * dv).numpy()
    return m


def _memory_plain(m, rows=None, state=None):
    rows, z = m.rows if rows is None else rows, m.z
    H, d, dv, T = m.H, m.d, m.dv, rows.shape[0]
    f = plain.silu if m.silu else (lambda x: x)
    q, k, v, g = np.split(rows, np.cumsum([H * d, H * d, H * dv]), axis=1)
    if m.log_decay is None:
        a = np.exp(plain.log_sigmoid(z + m.bias) / m.tau).reshape(T, H, d)
    else:
        a = np.broadcast_to(np.exp(m.log_decay)[None, :, None], (T, H, d))
    o, S = plain.recurrence(f(q).reshape(T, H, d) * m.q_scale, f(k).reshape(T, H, d), f(v).reshape(T, H, dv), a, state)
    o = plain.rms(o, m.eps).reshape(T, -1) if m.head else plain.rms(o.reshape(T, -1), m.eps)
    return o * m.norm * (plain.silu(g) if m.gate else plain.sigmoid(g)), S


def _memory_run(ops, m, rows, z, state, ctx, dtype):
    f = lambda x: None if x is None else dev(torch.from_numpy(np.asarray(x)).float())
    out = torch.full((rows.shape[0], m.H * m.dv), float("nan"), device="cuda", dtype=dtype)
    ops.linear_attention(f(rows).to(dtype), f(z), f(m.log_decay), f(m.bias), m.tau, f(m.norm), state, ctx, out, m.H, m.d, m.dv,
                         "silu" if m.silu else None, m.q_scale, "head" if m.head else "all",
                         "silu" if m.gate else "sigmoid", m.eps)
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("constant", [True, False])
@pytest.mark.parametrize("sizes", [(3, 48, 72), (2, 6, 5), (1, 64, 64), (3, 24, 40), (2, 130, 33), (1, 300, 16),
                                   (5, 16, 132), (2, 33, 64)])
def test_linear_attention_kernel(ops, dtype, constant, sizes):
    """Three requests of unequal length in portions of unequal size (within a chunk, one chunk and a
    token more, several), one of them token by token, in state slots that are not in order."""
    H, d, dv = sizes
    gen = torch.Generator().manual_seed(d + dv)
    flags = (constant, not constant, not constant)           # both forms of the norm and the gate
    lengths = {"a": 240, "b": 9, "c": 66}
    ms = {r: _memory(gen, H, d, dv, constant, *flags, n) for r, n in lengths.items()}
    base = ms["a"]
    for m in ms.values():
        m.bias, m.norm = base.bias, base.norm
    want = {r: _memory_plain(m) for r, m in ms.items()}
    state = torch.zeros(6, H * d * dv, device="cuda")
    state[4].fill_(3.0)                                      # never touched
    slot = {"a": 5, "b": 0, "c": 2}
    cuts = {"a": [65, 2, 1, 127, 45], "b": [1] * 9, "c": [2, 64]}
    done, got = {r: 0 for r in lengths}, {r: [] for r in lengths}
    for step in range(9):
        parts = [(r, cuts[r][step]) for r in ("b", "a", "c") if step < len(cuts[r])]
        parts.sort(key=lambda p: p[1] != 1)                  # single tokens first
        single = [p for p in parts if p[1] == 1]
        # empty requests and filling requests without a slot, as padded steps have
        layout = single + [(None, 1)] + parts[len(single):] + [(None, 0), (None, 70)]
        ctx, starts = step_context([(n, slot[r] if r else -1) for r, n in layout])
        rows, z = (None if x == "z" and constant else np.concatenate(
            [getattr(ms[r], x)[done[r]:done[r] + n] if r else np.full((n, getattr(base, x).shape[1]), 1e3)
             for r, n in layout]) for x in ("rows", "z"))
        out = _memory_run(ops, base, rows, z, state, ctx, dtype)
        for (r, n), a in zip(layout, starts):
            if r:
                got[r].append(out[a:a + n].cpu())
                done[r] += n
            else:
                assert float(out[a:a + n].abs().max() if n else 0.0) == 0.0
    for r in lengths:
        close(torch.cat(got[r]), want[r][0], dtype, bound=3e-5 if dtype == torch.float32 else None)
        S = want[r][1]
        # (activated keys and values of bfloat16 rows are rounded once more)
        loose = dtype == torch.bfloat16 and flags[0]
        close(state[slot[r]], S.reshape(-1), torch.float32, bound=1e-2 if loose else 3e-5, scale=max(1.0, float(np.abs(S).max())))
    assert float((state[4] - 3.0).abs().max()) == 0 and float(state[1].abs().max()) == 0


@pytest.mark.parametrize("dtype,sizes", [(torch.float32, (3, 40, 24)), (torch.bfloat16, (3, 48, 32)),
                                         (torch.bfloat16, (2, 128, 80)), (torch.bfloat16, (2, 20, 12))])
def test_decays_from_nothing_to_one(ops, dtype, sizes):
    """Decays that forget everything at once, beside decays that forget nothing, over many chunks: no
    infinity, no lost token.  Constant decays of 0 and 1, and decays by channel whose exponents
    reach some thousands within a chunk."""
    gen = torch.Generator().manual_seed(5)
    (H, d, dv), n = sizes, 400
    for constant in (True, False):
        m = _memory(gen, H, d, dv, constant, False, False, False, n)
        if constant:
            m.log_decay = np.array([-1e4, 0.0, np.log(0.5)])[:H]
        else:
            m.tau = 0.5
            z = m.z.reshape(n, H, d)
            z[:, :, ::3] = -150.0                            # forgets all
            z[:, :, 1::3] = 60.0                             # forgets nothing
            z[::50, :, 2::3] = -40.0                         # now and then
        want, S = _memory_plain(m)
        for cut in ([n], [64, 1, 2, 130] * 2 + [6], [1] * 30 + [n - 30]):
            state = torch.zeros(1, H * d * dv, device="cuda")
            outs, at = [], 0
            for c in cut:
                c = min(c, n - at)
                if c <= 0:
                    break
                ctx, _ = step_context([(c, 0)])
                outs.append(_memory_run(ops, m, m.rows[at:at + c], None if m.z is None else m.z[at:at + c], state, ctx, dtype).cpu())
                at += c
            got = torch.cat(outs)
            assert at == n
            close(got, want, dtype, bound=1e-4 if dtype == torch.float32 else None)
            close(state[0], S.reshape(-1), torch.float32, bound=1e-4)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_an_early_token_among_hundreds_is_not_lost(ops, dtype):
    """One early token's key and value are large and every decay is near one: it is seen by a query of
    each later chunk, in portions and in single tokens."""
    gen = torch.Generator().manual_seed(6)
    H, d, dv, n = 2, 16, 16, 330
    m = _memory(gen, H, d, dv, True, False, True, True, n)
    m.log_decay = np.log(np.array([0.9999, 0.999]))
    m.rows[:, H * d:2 * H * d + H * dv] *= 0.01
    m.rows[3, H * d:2 * H * d + H * dv] *= 3000.0
    m.rows = torch.from_numpy(m.rows).to(torch.bfloat16).double().numpy()
    want, _ = _memory_plain(m)
    without = m.rows.copy()
    without[3, H * d:2 * H * d] = 0.0
    assert np.abs(_memory_plain(m, without)[0][-1] - want[-1]).max() > 0.1     # to the last query
    for cut in ([n], [2, 63, 65, 200], [300] + [1] * 30):
        state, outs, at = torch.zeros(1, H * d * dv, device="cuda"), [], 0
        for c in cut:
            ctx, _ = step_context([(c, 0)])
            outs.append(_memory_run(ops, m, m.rows[at:at + c], None if m.z is None else m.z[at:at + c], state, ctx, dtype).cpu())
            at += c
        close(torch.cat(outs), want, dtype, bound=3e-5 if dtype == torch.float32 else None)


# ---- router -----------------------------------------------------------------------------------------

def test_router_weighs_with_the_chosen_logits_alone(ops):
    g = torch.Generator().manual_seed(2)
    for E, top, W, n in ((12, 3, 176, 50), (5, 1, 50, 9), (8, 8, 64, 20), (64, 6, 128, 33), (40, 33, 24, 5)):
        x = rnd(g, torch.bfloat16, n, W)
        router = rnd(g, torch.float32, E, W, std=4 * W ** -0.5)
        for xt in (torch.float32, torch.bfloat16):
            ids = torch.empty(n, top, dtype=torch.int32, device="cuda")
            wts = torch.empty(n, top, dtype=torch.float32, device="cuda")
            ops.moe_route(dev(x, xt), dev(router.float()), 1, 1, 2, 1e-20, ids, wts, score="softmax_chosen")
            for t in range(n):
                chosen, w = plain.route((router @ x[t]).numpy(), top)
                assert ids[t].tolist() == list(chosen), (E, t)
                assert np.allclose(wts[t].cpu().numpy(), w, rtol=2e-5, atol=1e-7)
    # logits so far apart that the softmax over all of them would be 0 for the second one chosen, and
    # equal logits: the lower index first
    logits = dev(torch.tensor([[-300.0, 0.0, -200.0, 0.0, -1e4]]))
    ids = torch.empty(1, 3, dtype=torch.int32, device="cuda")
    wts = torch.empty(1, 3, dtype=torch.float32, device="cuda")
    ops.moe_select(logits, 1, 1, 2, 1e-20, ids, wts, score="softmax_chosen")
    assert ids.tolist() == [[1, 3, 2]] and wts[0, :2].tolist() == [0.5, 0.5]


# ---- the engine -------------------------------------------------------------------------------------

_models = {}


def engine(folder, dtype):
    from rvllm_b200.engine import load_model
    if (folder, dtype) not in _models:
        _models[(folder, dtype)] = load_model(folder, dtype, "cuda")[0]
    return _models[(folder, dtype)]


def run_schedule(model, steps, page, slots=4, graphs=False):
    from rvllm_b200.engine import ModelRunner, make_cache
    cache = make_cache(model, page, schedules.tokens_held(steps, 64) // page, slots)
    runner = ModelRunner(model, cache, model.ops, use_graphs=graphs)
    got = schedules.replay(runner, steps)
    model.ops.check_status()
    assert not cache.requests and all(g.pool.in_use == 0 for g in cache.groups)
    return got, runner


_plain = {}


def compare(got, folder, cfg, reqs, dtype, share=0.04):
    """float32: every position within the bound.  bfloat16: a router score that is a close call
    may fall the other way after rounding and change a token's experts, which is no fault; so a
    few positions in a hundred may lie outside the bound."""
    over, total = [], 0
    for rid, ids in reqs.items():
        key = (folder, tuple(ids))
        if key not in _plain:
            _plain[key] = fk.plain_logits(folder, None, ids, cfg=cfg)
        ref = _plain[key]
        scale = float(ref.abs().max())
        for p in range(len(ids)):
            err = float((got[(rid, p)].double() - ref[p]).abs().max()) / scale
            total += 1
            if not err < BOUND[dtype]:
                over.append((rid, p, err))
    assert len(over) <= (0 if dtype == "float32" else share * total), (len(over), total, over[:5])


def _requests(vocab, lengths, seed):
    rng = random.Random(seed)
    return {f"q{i}": [rng.randrange(vocab) for _ in range(n)] for i, n in enumerate(lengths)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_every_cut_equals_plain(folders, name, dtype):
    """Whole prompts; a prompt then its last tokens one by one; portions down to two tokens;
    mixed batches of unequal requests on four slots, with more requests than slots, so that
    pages and slots are used again."""
    model = engine(folders[name], dtype)
    cfg = fk.config(name)
    reqs = _requests(cfg["vocab"], (130, 1, 2, 67, 200, 33, 64, 65), 3)
    f = folders[name]
    compare(run_schedule(model, schedules.whole(reqs), 16)[0], f, cfg, reqs, dtype)
    compare(run_schedule(model, schedules.tail_decode(reqs, 90), 8)[0], f, cfg, reqs, dtype)
    compare(run_schedule(model, schedules.portions(reqs), 16)[0], f, cfg, reqs, dtype)
    compare(run_schedule(model, schedules.portions(reqs, (64, 2, 100, 3)), 4)[0], f, cfg, reqs, dtype)
    for seed in (0, 1):
        compare(run_schedule(model, schedules.mixed(reqs, seed), 16)[0], f, cfg, reqs, dtype)


def _one_mechanism(tmp, which):
    """A model of one layer whose mixer is sharp (a large scale, large projections), so that a
    single lost or misplaced key changes the result by much more than the bound."""
    from rvllm_b200.config import config_from_dict
    from rvllm_b200.weights import write_random_model
    from rvllm_b200.weights.safetensors_io import SafetensorsFile, write_streamed
    if which == "lightning":
        layer = {"type": "lightning", "mlp": None, "mixer": fk._lightning(3, 40, 24)}
    else:
        layer = {"type": "parallel", "mlp": None,
                 "mixer": {"left": fk._left(6, 3, 32, 25, 6, 3.0, 40.0, fk._rot(20, 50.0, (3.0, 40, 6.0, 0.7))),
                           "right": fk._right(2, 24, 40, 5.0, 6)}}
    cfg = {"architecture": "Fekizen", "vocab": 150, "width": 72, "max_positions": 450, "norm": {"eps": 1e-5},
           "embedding": {"scale": 3.0}, "layers": [layer]}
    folder = write_random_model(os.path.join(tmp, which), config_from_dict(copy.deepcopy(cfg)), 7)
    path = os.path.join(folder, "model.safetensors")
    f = SafetensorsFile(path)
    tensors = {n: f.tensor(n).clone() for n in f.names()}
    del f
    quiet = {"left": ".right.out", "right": ".left.out"}.get(which)
    for n, t in tensors.items():                              # projections that give scores of size
        if n.endswith((".q", ".k", "embed")):
            tensors[n] = (t.float() * 6.0).to(t.dtype)
        if quiet and n.endswith(quiet):                       # the other branch does not show
            tensors[n] = torch.zeros_like(t)
    write_streamed(path, [(n, tuple(t.shape), t.dtype) for n, t in tensors.items()],
                   lambda n: tensors[n])
    return folder, cfg


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["left", "right", "lightning"])
def test_one_mechanism_alone_with_sharp_scores(tmp_path_factory, which, dtype):
    """Keys far away (hundreds of positions back), at page borders and in the first tokens,
    in prompts, in portions that begin inside a page, a block and a chunk, and in single tokens."""
    folder, cfg = _one_mechanism(str(tmp_path_factory.mktemp("one")), which)
    model = engine(folder, dtype)
    reqs = _requests(cfg["vocab"], (400, 63, 17), 11)
    ref = fk.plain_logits(folder, None, reqs["q0"], cfg=cfg)
    assert float(ref.abs().max()) > 0.05
    for steps, page in ((schedules.whole(reqs), 16), (schedules.tail_decode(reqs, 40), 8),
                        (schedules.portions(reqs, (15, 2, 17, 130, 3)), 16),
                        (schedules.mixed(reqs, 4), 4)):
        compare(run_schedule(model, steps, page)[0], folder, cfg, reqs, dtype, share=0.05)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D"])
def test_replayed_steps_equal_plain(folders, name, dtype):
    """The same with captured launch sequences: single-token steps and padded mixtures are
    replayed from graphs; requests come and go, so slots and pages are used again."""
    model = engine(folders[name], dtype)
    cfg = fk.config(name)
    reqs = _requests(cfg["vocab"], (90, 5, 41, 120, 33, 70, 18), 8)
    for steps, page in ((schedules.tail_decode(reqs, 40), 16), (schedules.mixed(reqs, 2), 8),
                        (schedules.mixed(reqs, 3, max_live=3, decode_tail=20), 16)):
        got, runner = run_schedule(model, steps, page, graphs=True)
        compare(got, folders[name], cfg, reqs, dtype)
        assert runner.graph_steps > 0


def test_long_decoding(folders):
    """600 tokens one by one after a short prompt, across many pages, blocks and splits, to the end
    of the position table."""
    model = engine(folders["B"], "float32")
    cfg = fk.config("B")
    reqs = _requests(cfg["vocab"], (700,), 6)
    got, _ = run_schedule(model, schedules.tail_decode(reqs, 680), 16, graphs=True)
    compare(got, folders["B"], cfg, reqs, "float32")


def test_a_batch_does_not_change_a_request(folders):
    """A request beside others gives what it gives alone, in the same cut."""
    model = engine(folders["A"], "float32")
    reqs = _requests(fk.config("A")["vocab"], (70, 31, 5), 12)
    alone, _ = run_schedule(model, schedules.whole({"q0": reqs["q0"]}), 16)
    steps = [{"step": 0, "entries": [{"id": r, "tokens": ids, "want": list(range(len(ids)))}
                                      for r, ids in reqs.items()], "end": list(reqs)}]
    together, _ = run_schedule(model, steps, 16)
    scale = max(float(alone[("q0", p)].abs().max()) for p in range(70))
    for p in range(70):
        assert float((alone[("q0", p)] - together[("q0", p)]).abs().max()) < 1e-5 * scale


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(folders, name):
    """Greedy tokens through `Generator` (scheduler, portions, preemption by a small pool) equal
    the plain implementation's argmax chain."""
    from rvllm_b200 import GenerateOptions, Generator
    rng = random.Random(9)
    cfg = fk.config(name)
    new = 20
    tensors = fk.read_tensors(folders[name])

    def plain_greedy(ids):
        """The argmax chain, or None when two logits on the way are too close to call."""
        ids = list(ids)
        for _ in range(new):
            row = fk.plain_logits(folders[name], name, ids, tensors=tensors)[-1]
            top = torch.topk(row, 2).values
            if float(top[0] - top[1]) < 1e-3 * float(row.abs().max()):
                return None
            ids.append(int(row.argmax()))
        return ids[-new:]

    prompts, want = [], []
    for n in (5, 37, 70):
        for attempt in range(20):
            p = [rng.randrange(cfg["vocab"]) for _ in range(n)]
            w = plain_greedy(p)
            if w is not None:
                prompts.append(p)
                want.append(w)
                break
    assert len(prompts) == 3
    gen = Generator.load(folders[name], dtype="float32")
    for opts in (GenerateOptions(max_tokens=new, block_size=16, stop_tokens=[]),
                 GenerateOptions(max_tokens=new, block_size=8, stop_tokens=[], prefill_chunk=7,
                                 max_batched_tokens=12),
                 GenerateOptions(max_tokens=new, block_size=8, stop_tokens=[], num_blocks=16,
                                 prefill_chunk=20)):
        assert gen.complete_batch(prompts, opts) == want


def test_command_line_and_trace_replay(folders, tmp_path):
    """The design through the programs a user starts: `rvllm random-model` writes a folder from a
    config.json, `rvllm cli` completes prompts of token ids, `bin/trace_run` replays steps from
    standard input and writes logits that equal the plain implementation's."""
    import json
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(fk.config("B")))
    folder = str(tmp_path / "model")
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "rvllm"), "random-model",
                        "--config", str(cfg_path), "--seed", "5", "--out", folder],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    tensors = fk.read_tensors(folder)
    prompt = [3, 1, 4, 1, 5, 9, 2, 6]
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "rvllm"), "cli", "--model", folder,
                        "--dtype", "float32", "--token-ids", "--prompt", " ".join(map(str, prompt)),
                        "--max-tokens", "5", "--block-size", "8"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    got = [int(t) for t in r.stdout.strip().splitlines()[0].split()]
    ids = list(prompt)
    for tok in got:                           # each token is the plain argmax at its place
        row = fk.plain_logits(folder, "B", ids, tensors=tensors)[-1]
        assert float(row.max() - row[tok]) < 1e-3 * float(row.abs().max())
        ids.append(tok)
    assert len(got) == 5
    reqs = _requests(fk.config("B")["vocab"], (70, 33, 90, 41, 12), 4)
    steps = schedules.mixed(reqs, seed=2)
    vocab = fk.config("B")["vocab"]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        cmd = [sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder,
               "--dtype", dtype, "--out", str(out), "--max-tokens",
               str(schedules.tokens_held(steps, 64))]
        r = subprocess.run(cmd, input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=900)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.split("\n") if l.startswith("done")] == \
            [f"done {s['step']}" for s in steps]
        got, pos = {}, {k: 0 for k in reqs}
        for s in steps:
            arr = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, vocab)
            k = 0
            for e in s["entries"]:
                for w in e["want"]:
                    got[(e["id"], pos[e["id"]] + w)] = torch.from_numpy(arr[k].copy())
                    k += 1
                pos[e["id"]] += len(e["tokens"])
            assert k == arr.shape[0]
        over, total = 0, 0
        for rid, ids in reqs.items():
            ref = fk.plain_logits(folder, "B", ids, tensors=tensors)
            for p in range(len(ids)):
                err = float((got[(rid, p)].double() - ref[p]).abs().max() / ref.abs().max())
                total += 1
                over += not err < BOUND[dtype]
        assert over <= (0 if dtype == "float32" else 0.04 * total), (dtype, over, total)
