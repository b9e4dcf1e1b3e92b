"""Buzinex on the GPU against the plain implementation: every mechanism alone (with inputs made so that a fault shows),
then whole models under every way of cutting the work, through the step function, the trace replay program and the
scheduler."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import buzinex_helpers as bh
import helpers
import plain_buzinex as plain

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 6e-5, "bfloat16": 6e-2}       # of the logits' spread over the vocabulary at that place (buzinex_helpers.relative)


def rounded(array, dtype):
    """float32 values that ``dtype`` holds exactly."""
    return torch.from_numpy(np.asarray(array, dtype=np.float32)).to(DTYPES[dtype]).float()


def dev(array, dtype=None):
    t = array if isinstance(array, torch.Tensor) else torch.from_numpy(np.ascontiguousarray(array))
    return (t.to(DTYPES[dtype]) if dtype else t).to(DEV)


def ints(values):
    return torch.tensor([int(v) for v in values], dtype=torch.int32, device=DEV)


def f64(t):
    return t.numpy().astype(np.float64)


def new_status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def drive(lengths, slots, cycle, step, limit=None, holdout=True):
    """Runs requests of the given lengths through ``step(pieces, slots)`` (pieces: request -> (from, to)) in portions that
    follow ``cycle``, several requests at a time and some left out of a step; what each step returned per request, in order."""
    done, got, k = {r: 0 for r in lengths}, {r: [] for r in lengths}, 0
    while any(done[r] < min(n, limit or n) for r, n in lengths.items()):
        pieces = {}
        for r, n in lengths.items():
            n = min(n, limit or n)
            if done[r] < n and not (holdout and len(lengths) > 1 and (r + k) % 3 == 0):
                pieces[r] = (done[r], done[r] + min(cycle[(k + r) % len(cycle)], n - done[r]))
        k += 1
        if not pieces:
            continue
        for r, rows in step(pieces, slots).items():
            got[r].append(rows)
            done[r] = pieces[r][1]
    return {r: np.concatenate(rows) for r, rows in got.items()}


def batch_context(pieces, slots):
    counts = [b - a for a, b in pieces.values()]
    return (SimpleNamespace(q_start=ints(np.concatenate([[0], np.cumsum(counts)])), max_q_len=max(counts),
                            seq_of_token=ints(np.repeat(np.arange(len(counts)), counts))),
            ints([slots[r] for r in pieces]), counts)


def split(rows, pieces, counts):
    out, at = {}, 0
    for r, n in zip(pieces, counts):
        out[r] = rows[at:at + n]
        at += n
    return out


# =============================================================================== mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [36, 64, 129])
def test_blends_with_the_row_before(dtype, width):
    """Portions down to one row, requests beside one another and left out of steps, slots that others used; the first row of a
    sequence blends with zeros, the last row of a portion is kept for the next one."""
    from sprout_lm_b200 import kernels
    rng = np.random.default_rng(width)
    parts = 5
    mu = rng.uniform(-0.2, 1.2, size=(parts, width)).astype(np.float32)
    lengths = dict(enumerate((70, 1, 9, 33)))
    data = {r: rounded(rng.normal(size=(n, width)), dtype) for r, n in lengths.items()}
    for cycle in ((100,), (2, 1, 5, 34, 3), (1,)):
        slots = {0: 2, 1: 0, 2: 4, 3: 1}
        state = torch.full((5, width), 7.0, dtype=torch.float32, device=DEV)
        for s in slots.values():
            state[s].zero_()
        status = new_status()

        def step(pieces, slots):
            ctx, slot_ids, counts = batch_context(pieces, slots)
            rows = dev(torch.cat([data[r][a:b] for r, (a, b) in pieces.items()]), dtype)
            out = torch.empty(rows.shape[0], parts * width, dtype=rows.dtype, device=DEV)
            kernels.token_blend(rows, dev(mu), out, ctx, SimpleNamespace(buffer=state, slots=slot_ids), status)
            return split(out.float().cpu().numpy().reshape(-1, parts, width), pieces, counts)
        got = drive(lengths, slots, cycle, step)
        for r in lengths:
            for s in range(parts):
                want = plain.blend_with_before(f64(data[r]), mu[s].astype(np.float64))
                assert (np.abs(got[r][:, s] - want) <= (2e-6 if dtype == "float32" else 5e-3) * (1 + np.abs(want))).all(), (r, s, cycle)
            assert np.array_equal(state[slots[r]].cpu().numpy(), data[r][-1].numpy())
        assert (state[3] == 7.0).all() and int(status.item()) == 0
    ctx, _, _ = batch_context({0: (0, 2)}, {0: 0})
    out = torch.empty(2, parts * width, dtype=DTYPES[dtype], device=DEV)
    kernels.token_blend(dev(data[0][:2], dtype), dev(mu), out, ctx, SimpleNamespace(buffer=state, slots=ints([5])), status)
    assert int(status.item()) == 1                                             # a slot outside the buffer is flagged, not touched


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(3, 6), (2, 11), (1, 40), (4, 64), (2, 128), (1, 300)])
def test_decay_with_bonus_whole_portions_and_single_tokens(sizes, dtype):
    """The recurrence whose output reads the state before the token: decays from almost none to almost everything, bonuses of both
    signs, long requests in chunks side by side, portions of changing size from states that are not zero, single tokens."""
    from sprout_lm_b200 import kernels
    H, D = sizes
    rng = np.random.default_rng(H * 1000 + D)
    lengths = dict(enumerate((300, 1, 129, 64, 5)))
    bias, bonus = np.linspace(-8.0, 1.5, H * D).astype(np.float32), rng.uniform(-2.0, 2.0, H * D).astype(np.float32)
    data, want = {}, {}
    for r, n in lengths.items():
        data[r] = {key: rounded(rng.normal(size=(n, H * D)), dtype) for key in ("r", "k", "v")}
        data[r]["z"] = torch.from_numpy(rng.normal(size=(n, H * D)).astype(np.float32))          # 32-bit on both paths
        d = {key: f64(v).reshape(n, H, D) for key, v in data[r].items()}
        w = np.exp(-np.exp(d["z"] + bias.reshape(H, D)))
        want[r] = plain.decay_with_bonus(d["r"], d["k"], d["v"], w, bonus.reshape(H, D).astype(np.float64))
    status = new_status()

    def stepper(state):
        def step(pieces, slots):
            ctx, slot_ids, counts = batch_context(pieces, slots)
            take = {key: dev(torch.cat([data[r][key][a:b] for r, (a, b) in pieces.items()]), None if key == "z" else dtype) for key in "rkvz"}
            o = torch.empty(take["r"].shape[0], H * D, dtype=torch.float32, device=DEV)
            kernels.gated_scan(take["r"], take["k"], take["v"], take["z"], dev(bias), ctx, SimpleNamespace(buffer=state, slots=slot_ids), o,
                               H, H, D, D, status, bonus=dev(bonus))
            return split(o.cpu().numpy().reshape(-1, H, D), pieces, counts)
        return step

    for label, cycle, slots in (("whole", (400,), {0: 4, 1: 0, 2: 5, 3: 2, 4: 1}), ("portions", (17, 2, 131, 1, 64, 3, 128), {0: 1, 1: 3, 2: 0, 3: 5, 4: 2}),
                                ("single", (1,), {0: 5, 1: 4, 2: 3, 3: 2, 4: 0})):
        state = torch.full((6, H, D, D), 7.0, dtype=torch.float32, device=DEV)
        for s in slots.values():
            state[s].zero_()
        got = drive(lengths, slots, cycle, stepper(state), limit=40 if label == "single" else None, holdout=label == "portions")
        for r, (o, S) in want.items():
            n = len(got[r])
            assert np.abs(got[r] - o[:n]).max() <= 3e-5 * max(1.0, np.abs(o).max()), (label, r, np.abs(got[r] - o[:n]).max())
            if n == len(o):
                assert np.abs(state[slots[r]].cpu().numpy() - S).max() <= 3e-5 * max(1.0, np.abs(S).max()), (label, r)
        assert (state[[s for s in range(6) if s not in slots.values()]] == 7.0).all()
    assert int(status.item()) == 0


def test_row_kernels():
    """RMS norms after a sublayer with the sum and the next norm in one launch, the buffer cleared behind it; the norm per head
    with a 32-bit gate beside 16-bit rows; tanh; scaled and capped logits."""
    from sprout_lm_b200 import kernels
    rng = np.random.default_rng(1)
    for width in (36, 128, 257, 768):
        x, y = (rng.normal(m, s, size=(5, width)).astype(np.float32) for m, s in ((0.5, 1.0), (-2.0, 3.0)))
        w1, w2 = (rng.uniform(0.3, 2.0, size=width).astype(np.float32) for _ in range(2))
        want = x + plain.rms_norm(y.astype(np.float64), w1, 1e-5)
        for dtype, tol in (("float32", 1e-5), ("bfloat16", 2e-2)):
            for clear in (False, True):
                got, buffer, h = dev(x.copy()), dev(y.copy()), torch.empty(5, width, dtype=DTYPES[dtype], device=DEV)
                kernels.norm_add(buffer, dev(w1), got, 1e-5, next_gain=dev(w2), h=h, rms=True, clear=clear)
                assert np.abs(got.cpu().numpy() - want).max() <= 5e-6
                assert np.abs(h.float().cpu().numpy() - plain.rms_norm(want, w2, 1e-5)).max() <= tol
                assert (buffer.cpu().numpy() == (0.0 if clear else y)).all()
    for heads, dim in ((3, 7), (2, 64)):
        o, gate = (rng.normal(size=(6, heads * dim)).astype(np.float32) for _ in range(2))
        weight = rng.uniform(0.3, 2.0, size=heads * dim).astype(np.float32)
        want = plain.unit_rms(o.astype(np.float64).reshape(6, heads, dim), 1e-6).reshape(6, -1) * weight * plain.silu(gate)
        for dtype, tol in (("float32", 4e-6), ("bfloat16", 2e-2)):
            out = torch.empty(6, heads * dim, dtype=DTYPES[dtype], device=DEV)
            kernels.gated_group_norm(dev(o), dev(gate), dev(weight), out, 1e-6, groups=heads, silu=True)
            assert np.abs(out.float().cpu().numpy() - want).max() <= tol
    z = rng.normal(0, 2.0, size=(9, 40)).astype(np.float32)
    for dtype, tol in (("float32", 1e-6), ("bfloat16", 4e-3)):
        out = torch.empty(9, 24, dtype=DTYPES[dtype], device=DEV)
        kernels.unit_act(dev(z)[:, 8:32], out, "tanh", gated=False)
        assert np.abs(out.float().cpu().numpy() - np.tanh(z[:, 8:32].astype(np.float64))).max() <= tol
    for cap, factor in ((3.0, 0.4), (0.0, -1.7), (50.0, 1.0)):
        got = dev(z.copy())
        kernels.softcap(got, cap, factor=factor)
        want = factor * z.astype(np.float64)
        assert np.abs(got.cpu().numpy() - (plain.soft_cap(want, cap) if cap else want)).max() <= 2e-6


@pytest.mark.parametrize("tokens", [1, 3, 16, 40, 130, 256, 300, 777])
@pytest.mark.parametrize("sizes", [(128, 72, (128, 128, 128, 24)), (64, 64, (256, 256, 40)), (96, 200, (384, 384, 384, 384, 100)),
                                   (40, 40, (56, 56, 24)), (33, 33, (128, 128, 9))])
def test_several_products_in_one_launch(sizes, tokens):
    """Matrices over inputs of their own: fused where the sizes allow it (inner sizes that are no multiple of 64, so that a block of
    columns reaches into the next input), a product each otherwise; the other inputs must not leak in."""
    from sprout_lm_b200.parts.linear import GroupedLinear
    inner, _, rows = sizes
    rng = np.random.default_rng(tokens + inner)
    for dtype in ("float32", "bfloat16"):
        weights = [rounded(rng.normal(0, 0.3, size=(n, inner)), dtype) for n in rows]
        a = rounded(rng.normal(size=(tokens, len(rows) * inner)) * np.repeat(10.0 ** np.arange(len(rows)), inner), dtype)
        status = new_status()
        layer = GroupedLinear([dev(w, dtype) for w in weights], status)
        assert (layer.fused is not None) == (dtype == "bfloat16" and inner % 8 == 0 and rows[0] % 128 == 0)
        got = layer.forward_float32(dev(a, dtype))
        for g, w in enumerate(weights):
            part = f64(a[:, g * inner:(g + 1) * inner])
            want = part @ f64(w).T
            assert got[g].dtype == torch.float32 and tuple(got[g].shape) == want.shape
            assert np.abs(got[g].cpu().numpy() - want).max() <= 2e-5 * np.abs(part).max() * inner ** 0.5, (dtype, g)
        assert int(status.item()) == 0


# ------------------------------------------------------------------------------- attention
def shuffled_pages(rng, contexts, page, spare=3):
    """(block tables with pages in shuffled order, pages in all)."""
    per = [-(-n // page) for n in contexts]
    total = sum(per) + spare
    order, table, at = rng.permutation(total), np.full((len(contexts), max(per)), -1, dtype=np.int32), 0
    for r, n in enumerate(per):
        table[r, :n] = order[at:at + n]
        at += n
    return table, total


# (heads, rank, rotated part, page, window or None, sink)
LATENT_CASES = [(3, 20, 6, 16, 5, True), (2, 14, 12, 8, 19, True), (1, 32, 8, 8, 1, True), (5, 48, 16, 8, 33, False), (8, 64, 16, 16, 70, True),
                (4, 96, 32, 16, 130, True), (16, 128, 64, 16, 64, True), (17, 256, 64, 16, 65, False), (8, 512, 64, 16, 200, True),
                (4, 64, 32, 32, None, True), (2, 160, 16, 16, 97, True)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", LATENT_CASES)
def test_latent_rows_over_a_window(dtype, case):
    """Contexts on both sides of page, window and 64-key borders; portions beside single rows, steps of single rows (whose keys
    several CTAs divide) laid out for shorter and longer contexts; pages that no row can see any more are gone from the
    tables and hold no numbers."""
    from sprout_lm_b200 import kernels
    H, rank, rot, page, window, has_sink = case
    rng = np.random.default_rng(H * 100 + rank)
    width, scale = rank + rot, 2.0 / np.sqrt(rank + rot)
    edges = {1, 2, page, page + 1, 63, 64, 65, 129, 200, 333, 700} | ({window - 1, window, window + 1, window + page, 2 * window + 3} if window else set())
    contexts = sorted(n for n in edges if n >= 1)[:16]
    q_lens = [min(n, q) for n, q in zip(contexts, (1, 1, 2, 1, 5, 1, 17, 1, 64, 1, 3, 1, 40, 1, 150, 1))]
    table, total = shuffled_pages(rng, contexts, page)
    cache = torch.full((total, 1, page, width), float("nan"), dtype=DTYPES[dtype], device=DEV)
    sink = rng.uniform(-1.0, 3.0, size=H).astype(np.float32) if has_sink else None
    wants, q_rows = [], []
    for r, (n, ql) in enumerate(zip(contexts, q_lens)):
        keys, q = rounded(rng.normal(size=(n, width)), dtype), rounded(rng.normal(size=(ql, H, width)), dtype)
        first_seen = 0 if window is None else max(0, n - ql - window + 1)
        for p in range(-(-n // page)):
            if (p + 1) * page <= first_seen:
                table[r, p] = -1                                              # given back: no row of this step sees it
                continue
            rows = keys[p * page:min(n, (p + 1) * page)]
            cache[table[r, p], 0, :len(rows)] = dev(rows, dtype)
            if p * page < first_seen:
                cache[table[r, p], 0, :first_seen - p * page] = float("nan")  # out of sight on a page that stays
        pk, pq, seen = f64(keys), f64(q), plain.visible(n, window)[n - ql:]
        out = np.zeros((ql, H, rank))
        for h in range(H):
            s = np.where(seen, plain.latent_scores(pq[:, h, :rank], pq[:, h, rank:], pk[:, :rank], pk[:, rank:], scale), -np.inf)
            out[:, h] = plain.softmax_rows(s, None if sink is None else sink[h]) @ pk[:, :rank]
        wants.append(out.reshape(ql, -1))
        q_rows.append(q.reshape(ql, -1))
    starts = np.concatenate([[0], np.cumsum(q_lens)])
    q_all, want = dev(torch.cat(q_rows), dtype), np.concatenate(wants)
    positions = np.concatenate([np.arange(n - ql, n) for n, ql in zip(contexts, q_lens)])
    status = new_status()
    tol = 3e-5 if dtype == "float32" else 3e-2

    def run(sel, planned):
        rows = np.concatenate([np.arange(starts[r], starts[r + 1]) for r in sel])
        counts = [q_lens[r] for r in sel]
        ctx = SimpleNamespace(q_start=ints(np.concatenate([[0], np.cumsum(counts)])), positions=ints(positions[rows]), num_seqs=len(sel),
                              seq_of_token=ints(np.repeat(np.arange(len(sel)), counts)), context_lens=ints([contexts[r] for r in sel]),
                              max_q_len=max(counts), planned_context=planned, max_context=max(contexts[r] for r in sel))
        view = SimpleNamespace(k=cache, block_table=dev(table[sel]), page_tokens=page, write=False)
        out = torch.empty(len(rows), H * rank, dtype=DTYPES[dtype], device=DEV)
        kernels.latent_attention(q_all[rows].contiguous(), view, ctx, None if sink is None else dev(sink), out, H, rank, scale, status,
                                 window=window or 0)
        err = np.abs(out.float().cpu().numpy() - want[rows]).max()
        assert err <= tol, (sel, planned, err)
    everyone = list(range(len(contexts)))
    singles = [r for r in everyone if q_lens[r] == 1]
    run(everyone, max(contexts))
    for planned in (0, 16, 4096):
        run(singles, planned)
    run(singles[-1:], contexts[singles[-1]])
    assert int(status.item()) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_latent_row_decides(dtype):
    """One row's score stands out among hundreds: just inside and just outside the window, far back without one, at page
    borders and at the token itself, in portions and single rows; and a sink that takes everything or nothing."""
    from sprout_lm_b200 import kernels
    H, rank, rot, page, window, n = 4, 64, 16, 16, 96, 401
    width = rank + rot
    rng = np.random.default_rng(9)
    table, total = shuffled_pages(rng, [n], page)
    status = new_status()
    direction = rng.normal(size=width)
    direction /= np.linalg.norm(direction)
    for place, size, seen in ((n - 96, window, True), (n - 97, window, False), (n - 1, window, True), (n - 1, 1, True), (n - 2, 1, False),
                              (0, None, True), (0, n, True), (0, n - 1, False), (15, None, True), (16, None, True), (304, window, False),
                              (319, window, True), (320, 81, True), (320, 80, False)):
        keys, q = rng.normal(0, 0.05, size=(n, width)), rng.normal(0, 0.05, size=(n, H, width))
        keys[place] = direction * 6.0
        q[n - 1] = direction * 6.0
        keys_t, q_t = rounded(keys, dtype), rounded(q, dtype)
        cache = torch.zeros((total, 1, page, width), dtype=DTYPES[dtype], device=DEV)
        for p in range(-(-n // page)):
            rows = keys_t[p * page:(p + 1) * page]
            cache[table[0, p], 0, :len(rows)] = dev(rows, dtype)
        view = SimpleNamespace(k=cache, block_table=dev(table), page_tokens=page, write=False)
        for ql in (1, 2, 23):
            ctx = SimpleNamespace(q_start=ints([0, ql]), positions=ints(range(n - ql, n)), num_seqs=1, seq_of_token=ints([0] * ql),
                                  context_lens=ints([n]), max_q_len=ql, planned_context=n, max_context=n)
            out = torch.empty(ql, H * rank, dtype=DTYPES[dtype], device=DEV)
            kernels.latent_attention(dev(q_t[n - ql:].reshape(ql, -1), dtype), view, ctx, None, out, H, rank, 0.5, status, window=size or 0)
            last = out[-1].float().cpu().numpy().reshape(H, rank)
            near = np.abs(last - keys_t[place, :rank].numpy()).max() < 0.05
            assert near == seen, (place, size, ql)
            for level, share in ((60.0, 0.0), (-60.0, 1.0)):
                kernels.latent_attention(dev(q_t[n - ql:].reshape(ql, -1), dtype), view, ctx, torch.full((H,), level, device=DEV), out, H, rank,
                                         0.5, status, window=size or 0)
                with_sink = out[-1].float().cpu().numpy().reshape(H, rank)
                assert np.abs(with_sink - share * last).max() < 1e-2, (place, size, ql, level)
    assert int(status.item()) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", [(6, 3, 9, 11, 16, 0.9, 3, 7.0), (4, 4, 16, 24, 8, -0.2, 20, 9.0), (3, 1, 32, 32, 8, 0.9, 64, 6.0),
                                  (8, 2, 64, 64, 16, 0.35, 50, 12.0), (2, 2, 64, 128, 16, 0.15, 7, 30.0), (6, 1, 128, 128, 16, 0.5, 256, 20.0),
                                  (4, 2, 48, 48, 16, 0.4, 1, 15.0)])
def test_attention_with_growing_queries_and_capped_scores(dtype, case):
    """Query and key norms, the growth of a query with its position (on both sides of every step of it), append and capped
    attention together, contexts on both sides of page and 64-key borders, portions beside single queries."""
    from sprout_lm_b200 import kernels
    H, G, dim, vdim, page, coef, every, cap = case
    rng = np.random.default_rng(H * 10 + dim)
    eps, scale = 1e-5, 2.0 / np.sqrt(dim)
    contexts = sorted({1, 2, page, page + 1, 64, 65, 129, 300, max(1, every - 1), every, every + 1, 3 * every})
    q_lens = [min(n, q) for n, q in zip(contexts, (1, 1, 2, 1, 5, 1, 17, 1, 64, 1, 3, 1))]
    table, total = shuffled_pages(rng, contexts, page)
    k_cache = torch.full((total, G, page, dim), float("nan"), dtype=DTYPES[dtype], device=DEV)
    v_cache = torch.full((total, G, page, vdim), float("nan"), dtype=DTYPES[dtype], device=DEV)
    qw, kw = (rng.uniform(0.4, 1.8, size=dim).astype(np.float32) for _ in range(2))
    status, wants, q_rows = new_status(), [], []
    for r, (n, ql) in enumerate(zip(contexts, q_lens)):
        q, k, v = (rounded(rng.normal(size=(n, heads, d)), dtype) for heads, d in ((H, dim), (G, dim), (G, vdim)))
        rows = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], dim=1)
        rows = dev(torch.nn.functional.pad(rows, (0, -rows.shape[1] % 8)), dtype)
        kernels.rope_maps_append(rows, ints(range(n)), ints([r] * n), dev(table), None, None, k_cache, v_cache, H, G, 1, dim, vdim, page, True,
                                 status, q_weight=dev(qw), k_weight=dev(kw), weight_eps=eps, growth=(coef, every))
        pq = plain.rms_norm(f64(q), qw, eps) * plain.query_growth(np.arange(n), coef, every)[:, None, None]
        pk, pv, seen = plain.rms_norm(f64(k), kw, eps), f64(v), plain.visible(n)[n - ql:]
        got_q = rows[:, :H * dim].float().cpu().numpy().reshape(n, H, dim)
        assert (np.abs(got_q - pq) <= (1e-5 if dtype == "float32" else 5e-3) * (1 + np.abs(pq))).all(), n
        out = np.zeros((ql, H, vdim))
        for h in range(H):
            g = h // (H // G)
            s = plain.soft_cap(pq[n - ql:, h] @ pk[:, g].T * scale, cap)
            out[:, h] = plain.softmax_rows(np.where(seen, s, -np.inf)) @ pv[:, g]
        wants.append(out.reshape(ql, -1))
        q_rows.append(rows[n - ql:, :H * dim])
    starts = np.concatenate([[0], np.cumsum(q_lens)])
    q_all, want = torch.cat(q_rows), np.concatenate(wants)
    positions = np.concatenate([np.arange(n - ql, n) for n, ql in zip(contexts, q_lens)])

    def run(sel):
        rows = np.concatenate([np.arange(starts[r], starts[r + 1]) for r in sel])
        counts = [q_lens[r] for r in sel]
        ctx = SimpleNamespace(q_start=ints(np.concatenate([[0], np.cumsum(counts)])), positions=ints(positions[rows]),
                              seq_of_token=ints(np.repeat(np.arange(len(sel)), counts)), max_q_len=max(counts),
                              planned_context=max(contexts[r] for r in sel), max_context=max(contexts))
        view = SimpleNamespace(k=k_cache, v=v_cache, block_table=dev(table[sel]), page_tokens=page, write=False)
        wide = torch.zeros(len(rows), -(-H * dim // 8) * 8, dtype=DTYPES[dtype], device=DEV)
        wide[:, :H * dim] = q_all[rows]
        out = torch.empty(len(rows), H * vdim, dtype=DTYPES[dtype], device=DEV)
        kernels.multimap_attention(wide[:, :H * dim], view, ctx, out, H, G, 1, dim, vdim, scale, 0.0, 0.0, 1.0, status, softcap=cap)
        err = np.abs(out.float().cpu().numpy() - want[rows]).max()
        assert err <= (4e-5 if dtype == "float32" else 6e-2), (sel, err)
    run(list(range(len(contexts))))
    run([r for r, n in enumerate(q_lens) if n == 1])
    assert int(status.item()) == 0


# =============================================================================== whole models
@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    base = tmp_path_factory.mktemp("buzinex")
    return {name: bh.make_model_dir(base, name) for name in bh.CONFIGS}


def make_requests(name, seed, lengths):
    vocab = bh.CONFIGS[name][0]["vocab"]
    rng = np.random.default_rng(seed)
    return {f"r{i}": helpers.random_tokens(rng, n, vocab) for i, n in enumerate(lengths)}


def make_runner(model_dir, dtype, pages, page_tokens, requests=4):
    from sprout_lm_b200.engine.step import ModelRunner
    from sprout_lm_b200.models import load_model
    model = load_model(model_dir, dtype=DTYPES[dtype])
    return ModelRunner(model, num_pages=pages, page_tokens=page_tokens, max_requests=requests, prefix_caching=False)


def test_layers_one_by_one(model_dirs):
    """The stream after every layer in 32-bit, so that a fault names its layer; the same with every block making its own
    first norm and with a block making the next one's."""
    from sprout_lm_b200.engine.batch import StepEntry
    for name, directory in model_dirs.items():
        config, tensors = bh.plain_model(directory)
        tokens = make_requests(name, 1, [41])["r0"]
        _, want = plain.forward(config, tensors, tokens, return_layers=True)
        for handed_on in (False, True):
            runner = make_runner(directory, "float32", 8, bh.CONFIGS[name][2])
            seen = []
            for block in runner.model.blocks:
                def wrapped(x, *args, _inner=block.forward, **more):
                    primed = _inner(x, *args, **more)
                    seen.append(x.clone())
                    return primed if handed_on else None
                block.forward = wrapped
            seq = runner.new_sequence()
            assert runner.reserve(seq, len(tokens))
            runner.step([StepEntry(seq, tokens, [0])])
            assert len(seen) == len(want)
            for i, (got, expected) in enumerate(zip(seen, want)):
                assert np.abs(got.cpu().numpy() - expected).max() <= 3e-5 * max(1.0, np.abs(expected).max()), (name, "layer", i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_all_cuttings_in_process(model_dirs, name, dtype):
    """Whole, tail decoded token by token (140 tokens: every window of the models passes over decoded tokens), portions
    down to two tokens, mixed batches with pages and state slots used again: against the plain implementation, and in 32-bit
    equal to one another to rounding."""
    page = bh.CONFIGS[name][2]
    requests = make_requests(name, 11, [5, 17, 33, 70, 170, 1, 40])
    plans = {
        "whole": helpers.plan_whole(requests),
        "tail": helpers.plan_tail_decode(requests, tail=140),
        "portions": helpers.plan_portions(requests),
        "mixed": helpers.plan_mixed(requests, np.random.default_rng(5)),
    }
    results = {}
    for label, plan in plans.items():
        budget = helpers.live_token_budget(plan, requests)
        runner = make_runner(model_dirs[name], dtype, budget // page, page, requests=4)
        got = results[label] = helpers.run_plan_in_process(runner, plan)
        assert len(got) == sum(len(t) for t in requests.values())
        worst = bh.compare(model_dirs[name], requests, got, TOL[dtype], f"{name}/{dtype}/{label}", page, rounded=dtype == "bfloat16")
        print(f"{name}/{dtype}/{label}: worst difference {worst:.2e}")
        runner.manager.check_invariants()
        for pool in runner.manager.pools:
            assert len(pool.free) == pool.num_pages                                           # every page came back
        assert len(runner.manager._free_state) == 4                                           # and every state slot
    if dtype == "float32":
        for label in ("tail", "portions", "mixed"):
            for place, row in results["whole"].items():
                assert np.abs(row - results[label][place]).max() <= 1e-4 * max(1.0, np.abs(row).max()), \
                    f"{name}: {label} differs from whole at {place}"


def test_long_context_and_long_decoding(model_dirs):
    """A prompt of several hundred tokens in uneven portions, then 140 tokens decoded one by one, in both dtypes: slow decays,
    windows that are no multiple of a page with pages given back, keys many pages back in the layers that see everything."""
    for name, page, pages in (("B", 8, 90), ("C", 16, 45)):
        requests = make_requests(name, 21, [670])
        plan = helpers.plan_portions(requests, sizes=(130, 2, 127, 3, 64, 100, 2, 97, 5) + (1,) * 140)
        for dtype in ("float32", "bfloat16"):
            runner = make_runner(model_dirs[name], dtype, pages, page)
            got = helpers.run_plan_in_process(runner, plan)
            bh.compare(model_dirs[name], requests, got, TOL[dtype], f"long/{name}/{dtype}", page, rounded=dtype == "bfloat16")


def test_a_whole_batch_of_long_prompts(model_dirs):
    """More tokens in a step than the products' small-batch forms take, several requests at once, chunks of the recurrence side by
    side."""
    name = "C"
    requests = make_requests(name, 23, [200, 130, 97])
    for dtype in ("float32", "bfloat16"):
        runner = make_runner(model_dirs[name], dtype, 40, 16)
        seqs = {rid: runner.new_sequence() for rid in requests}
        from sprout_lm_b200.engine.batch import StepEntry
        for rid, tokens in requests.items():
            assert runner.reserve(seqs[rid], len(tokens))
        rows = runner.step([StepEntry(seqs[rid], tokens, list(range(len(tokens)))) for rid, tokens in requests.items()]).cpu().numpy()
        runner.check_status()
        places = [(rid, pos) for rid, tokens in requests.items() for pos in range(len(tokens))]
        bh.compare(model_dirs[name], requests, dict(zip(places, rows)), TOL[dtype], f"batch/{dtype}", 16, rounded=dtype == "bfloat16")


def test_trace_replay_program(model_dirs, tmp_path):
    """bin/trace_run picks the model class by config.json and replays a mixed plan with four state slots."""
    name = "B"
    requests = make_requests(name, 13, [9, 40, 70, 23, 31, 12])
    plan = helpers.plan_mixed(requests, np.random.default_rng(2))
    budget = helpers.live_token_budget(plan, requests)
    vocab = bh.CONFIGS[name][0]["vocab"]
    for dtype in ("float32", "bfloat16"):
        got = helpers.run_plan_with_trace_run(model_dirs[name], dtype, plan, tmp_path / dtype, budget, vocab=vocab)
        bh.compare(model_dirs[name], requests, got, TOL[dtype], f"trace/{dtype}", 16, rounded=dtype == "bfloat16")


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_scheduler(model_dirs, name):
    """generate(): continuous batching, chunked prefill and captured decode steps; in 32-bit the tokens are the plain
    implementation's, in bfloat16 every token is within bfloat16's reach of the plain choice."""
    from sprout_lm_b200 import generate, load_model
    config, tensors = bh.plain_model(model_dirs[name])
    rng = np.random.default_rng(7)
    prompts = [helpers.random_tokens(rng, n, config["vocab"]) for n in (3, 19, 44)]
    for dtype in ("float32", "bfloat16"):
        results = generate(load_model(model_dirs[name], dtype=dtype), prompts, max_new_tokens=12, ignore_eos=True)
        for prompt, result in zip(prompts, results):
            assert len(result["output"]) == 12
            if dtype == "float32":
                assert result["output"] == bh.plain_greedy(model_dirs[name], prompt, 12)
            history = list(prompt)
            for token in result["output"]:
                row = plain.forward(config, tensors, history)[-1]
                spread = float(np.sqrt(np.mean((row - row.mean()) ** 2)))
                assert row[token] >= row.max() - (1e-4 if dtype == "float32" else 4 * TOL["bfloat16"]) * spread, (name, dtype, len(history))
                history.append(token)


def test_device_side_decode_loop(model_dirs):
    """Decode steps that run back to back on the device, from captured graphs: the states and windows move on without the host."""
    from sprout_lm_b200.engine.batch import StepEntry
    name = "A"
    directory, page = model_dirs[name], bh.CONFIGS[name][2]
    config, _ = bh.plain_model(directory)
    rng = np.random.default_rng(12)
    prompts = [helpers.random_tokens(rng, n, config["vocab"]) for n in (6, 21)]
    runner = make_runner(directory, "float32", 16, page)
    seqs = [runner.new_sequence() for _ in prompts]
    for seq, prompt in zip(seqs, prompts):
        assert runner.reserve(seq, len(prompt))
    first = runner.step_and_sample([StepEntry(s, p, [len(p) - 1]) for s, p in zip(seqs, prompts)], [0.0, 0.0], [0.0, 0.0])
    loop = runner.decode_loop([StepEntry(s, [t], [0]) for s, t in zip(seqs, first)], [0.0, 0.0], [0.0, 0.0], 9)
    loop.run(8)
    history = loop.finish().numpy()
    runner.check_status()
    for i, prompt in enumerate(prompts):
        assert [first[i], *history[:, i].tolist()] == bh.plain_greedy(directory, prompt, len(history) + 1)


def test_scheduler_under_page_pressure(model_dirs):
    """A pool smaller than the requests together: a preempted request gives its state slot back and recomputes its state
    from the start; the greedy tokens stay the plain implementation's."""
    from sprout_lm_b200 import EngineOptions, generate, load_model
    name = "A"
    config, _ = bh.plain_model(model_dirs[name])
    rng = np.random.default_rng(8)
    prompts = [helpers.random_tokens(rng, n, config["vocab"]) for n in (30, 41, 26, 35)]
    model = load_model(model_dirs[name], dtype="float32")
    options = EngineOptions(block_size=8, num_blocks=14, max_sequences=4, max_batch_tokens=24, prefill_chunk_size=7)
    results = generate(model, prompts, max_new_tokens=10, ignore_eos=True, options=options)
    for prompt, result in zip(prompts, results):
        assert result["output"] == bh.plain_greedy(model_dirs[name], prompt, 10)
