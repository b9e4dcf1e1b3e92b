"""Zevedra on the GPU against the plain implementation: every mechanism alone (with inputs made so that a fault shows),
then whole models under every way of cutting the work, through the step function, the trace replay program and the
scheduler."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import helpers
import plain_zevedra as plain
import zevedra_helpers as zh

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 6e-5, "bfloat16": 6e-2}       # of the logits' spread over the vocabulary at that place (zevedra_helpers.relative)


def rounded(array, dtype):
    """float32 values that ``dtype`` holds exactly."""
    return torch.from_numpy(np.asarray(array, dtype=np.float32)).to(DTYPES[dtype]).float()


def dev(array, dtype=None):
    t = array if isinstance(array, torch.Tensor) else torch.from_numpy(np.ascontiguousarray(array))
    return (t.to(DTYPES[dtype]) if dtype else t).to(DEV)


def f32(array):
    return dev(np.asarray(array, dtype=np.float32))


def ints(values):
    return torch.tensor([int(v) for v in values], dtype=torch.int32, device=DEV)


def f64(t):
    return t.numpy().astype(np.float64)


def new_status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


# =============================================================================== mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_token_pair_rows(dtype):
    """The last two tokens choose a row: across portions, beside other requests, in slots that other requests used before,
    for the first token of a sequence, and with products that need more than 31 bits."""
    from sprout_lm_b200 import kernels
    rng = np.random.default_rng(0)
    vocab, width, buckets, mul_prev, mul_cur, scale = 60000, 20, 89, 1_900_000_011, 1_300_000_021, 2.5
    table, pairs = rounded(rng.normal(size=(vocab, width)), dtype), rounded(rng.normal(size=(buckets + 1, width)), dtype)
    config = {"embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}
    w = {"embed": f64(table), "bigram": f64(pairs)}
    requests = {r: [int(t) for t in rng.integers(0, vocab, size=n)] for r, n in enumerate((1, 9, 30, 2, 17))}
    status, state = new_status(), torch.full((6, 1), 12345, dtype=torch.int32, device=DEV)
    slots, done, got, k = {0: 5, 1: 0, 2: 3, 3: 1, 4: 2}, {r: 0 for r in requests}, {r: [] for r in requests}, 0
    while any(done[r] < len(t) for r, t in requests.items()):
        pieces = {r: min((3, 1, 2, 8)[(k + r) % 4], len(t) - done[r]) for r, t in requests.items() if done[r] < len(t) and (r + k) % 3}
        k += 1
        if not pieces:
            continue
        tokens, positions, seqs = [], [], []
        for i, (r, n) in enumerate(pieces.items()):
            tokens += requests[r][done[r]:done[r] + n]
            positions += range(done[r], done[r] + n)
            seqs += [i] * n
        ctx = SimpleNamespace(token_ids=ints(tokens), positions=ints(positions), seq_of_token=ints(seqs),
                              q_start=ints(np.concatenate([[0], np.cumsum(list(pieces.values()))])))
        out = torch.empty(len(tokens), width, dtype=torch.float32, device=DEV)
        view = SimpleNamespace(buffer=state, slots=ints([slots[r] for r in pieces]))
        kernels.embed_pairs(dev(table, dtype), dev(pairs, dtype), ctx, view, out, scale, mul_prev, mul_cur, status)
        rows, at = out.cpu().numpy(), 0
        for r, n in pieces.items():
            got[r].append(rows[at:at + n])
            at += n
            done[r] += n
    for r, tokens in requests.items():
        assert np.abs(np.concatenate(got[r]) - plain.embed(config, w, np.array(tokens))).max() <= 2e-6, r
        assert int(state[slots[r]].item()) == tokens[-1]
    assert int(state[4].item()) == 12345 and int(status.item()) == 0
    ctx = SimpleNamespace(token_ids=ints([vocab]), positions=ints([0]), seq_of_token=ints([0]), q_start=ints([0, 1]))
    kernels.embed_pairs(dev(table, dtype), dev(pairs, dtype), ctx, SimpleNamespace(buffer=state, slots=ints([4])), out[:1], scale, 1, 1, status)
    assert int(status.item()) == 2                                           # a token beyond the table is flagged, not read


def test_row_kernels():
    """Two outputs normed over the width and added; a norm per head without a gate; a norm with one number."""
    from sprout_lm_b200 import kernels
    from sprout_lm_b200.parts import build_part
    from sprout_lm_b200.config.specs import PartSpec
    rng = np.random.default_rng(1)
    for width in (36, 257, 1030):
        x, y1, y2 = (rng.normal(0, s, size=(5, width)).astype(np.float32) for s in (1.0, 3.0, 0.01))
        w1, w2 = (rng.uniform(0.3, 2.0, size=width).astype(np.float32) for _ in range(2))
        got = dev(x.copy())
        kernels.rms_pair_add(dev(y1), dev(y2), dev(w1), dev(w2), got, 1e-5, -0.35)
        want = x - 0.35 * (plain.rms_norm(y1.astype(np.float64), w1, 1e-5) + plain.rms_norm(y2.astype(np.float64), w2, 1e-5))
        assert np.abs(got.cpu().numpy() - want).max() <= 4e-6
        norm = build_part("norm", PartSpec("rmsnorm", {"size": width, "eps": 1e-5, "name": "n", "suffix": "", "one_number": True}))
        assert norm.tensor_decls()[0].shape == ()
        norm.load(SimpleNamespace(vector=lambda name: torch.tensor(1.7, device=DEV), runtime=SimpleNamespace(dtype=torch.float32)))
        assert np.abs(norm.forward(dev(x)).cpu().numpy() - plain.rms_norm(x.astype(np.float64), 1.7, 1e-5)).max() <= 4e-6
    for heads, vdim in ((3, 7), (2, 64)):
        o = rng.normal(size=(6, heads, vdim)).astype(np.float32)
        weight = rng.uniform(0.3, 2.0, size=vdim).astype(np.float32)
        want = plain.rms_norm(o.astype(np.float64), weight, 1e-6).reshape(6, -1)
        for dtype, tol in (("float32", 4e-6), ("bfloat16", 2e-2)):
            out = torch.empty(6, heads * vdim, dtype=DTYPES[dtype], device=DEV)
            kernels.gated_group_norm(dev(o.reshape(6, -1)), None, dev(weight), out, 1e-6, groups=heads)
            assert np.abs(out.float().cpu().numpy() - want).max() <= tol


# ------------------------------------------------------------------------------- recurrences
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
    return (SimpleNamespace(q_start=ints(np.concatenate([[0], np.cumsum(counts)])), max_q_len=max(counts)),
            ints([slots[r] for r in pieces]), counts)


def split(rows, pieces, counts):
    out, at = {}, 0
    for r, n in zip(pieces, counts):
        out[r] = rows[at:at + n]
        at += n
    return out


DELTA_SIZES = [(3, 1, 7, 5), (2, 2, 4, 11), (4, 2, 16, 24), (1, 1, 20, 16), (4, 1, 48, 64), (2, 2, 64, 32), (2, 1, 128, 128), (1, 1, 200, 40),
               (2, 2, 256, 20), (8, 4, 32, 100)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", DELTA_SIZES)
def test_delta_rule_whole_portions_and_single_tokens(sizes, dtype):
    """The recurrence against float64: requests of unequal length in one batch (chunked, and walked token by token), portions
    of changing size from states that are not zero in slots that were used before, single tokens; decays from almost none to
    almost everything, keys that repeat (so that the write of the difference matters), heads that share keys."""
    from sprout_lm_b200 import kernels
    H, G, D, V = sizes
    rng = np.random.default_rng(H * 1000 + D)
    lengths = dict(enumerate((200, 1, 129, 64, 5, 65)))
    a_log, dt_bias = np.linspace(-5.0, 1.0, H).astype(np.float32), rng.uniform(-2.0, 1.0, H).astype(np.float32)
    data, want = {}, {}
    for r, n in lengths.items():
        few = rng.normal(size=(4, G * D))                                      # a handful of directions come again and again
        k = few[rng.integers(0, 4, size=n)] + 0.3 * rng.normal(size=(n, G * D))
        data[r] = {key: rounded(v, dtype) for key, v in (("q", rng.normal(size=(n, G * D))), ("k", k), ("v", rng.normal(size=(n, H * V))),
                                                         ("b", rng.normal(0, 2.0, size=(n, H))), ("a", rng.normal(0, 2.0, size=(n, H))))}
        d = {key: f64(v) for key, v in data[r].items()}

        def unit(x):
            x = x.reshape(n, G, D)
            return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)
        g = np.exp(-np.exp(a_log.astype(np.float64)) * plain.softplus(d["a"] + dt_bias))
        want[r] = plain.delta_rule(unit(d["q"]) * D ** -0.5, unit(d["k"]), d["v"].reshape(n, H, V), g, plain.sigmoid(d["b"]))
    status = new_status()

    def stepper(state):
        def step(pieces, slots):
            ctx, slot_ids, counts = batch_context(pieces, slots)
            rows = dev(torch.cat([torch.cat([data[r][key][a:b] for key in ("q", "k", "v", "b", "a")], dim=1) for r, (a, b) in pieces.items()]), dtype)
            at = 2 * G * D + H * V
            o = torch.empty(rows.shape[0], H * V, dtype=torch.float32, device=DEV)
            kernels.delta_rule(rows[:, :G * D], rows[:, G * D:2 * G * D], rows[:, 2 * G * D:at], rows[:, at:at + H], rows[:, at + H:],
                               dev(a_log), dev(dt_bias), ctx, SimpleNamespace(buffer=state, slots=slot_ids), o, H, G, D, V, status,
                               q_scale=D ** -0.5)
            return split(o.cpu().numpy().reshape(-1, H, V), pieces, counts)
        return step

    def fresh(slots):
        state = torch.full((8, H, D, V), 7.0, dtype=torch.float32, device=DEV)     # rubbish from earlier use
        for s in slots.values():
            state[s].zero_()
        return state

    def check(got, state, slots, label):
        for r, (o, S) in want.items():
            n = len(got[r])
            assert np.abs(got[r] - o[:n]).max() <= 3e-5 * max(1.0, np.abs(o).max()), (label, r, np.abs(got[r] - o[:n]).max())
            if n == len(o):
                assert np.abs(state[slots[r]].cpu().numpy() - S).max() <= 3e-5 * max(1.0, np.abs(S).max()), (label, r)
        untouched = [s for s in range(8) if s not in slots.values()]
        assert (state[untouched] == 7.0).all(), label

    slots = {0: 4, 1: 0, 2: 6, 3: 2, 4: 1, 5: 7}
    state = fresh(slots)
    check(stepper(state)({r: (0, n) for r, n in lengths.items()}, slots), state, slots, "whole")
    slots = {0: 1, 1: 3, 2: 0, 3: 5, 4: 2, 5: 6}
    state = fresh(slots)
    check(drive(lengths, slots, (17, 2, 131, 1, 64, 3, 24, 23), stepper(state)), state, slots, "portions")
    state = fresh(slots)
    check(drive(lengths, slots, (2, 9, 23, 1, 16), stepper(state)), state, slots, "short portions")
    state = fresh(slots)
    check(drive(lengths, slots, (1,), stepper(state), limit=40, holdout=False), state, slots, "single tokens")
    assert int(status.item()) == 0
    bad = fresh({})
    ctx, _, _ = batch_context({0: (0, 1)}, {0: 0})
    o = torch.empty(1, H * V, dtype=torch.float32, device=DEV)
    row = torch.zeros(1, 2 * G * D + H * V + 2 * H, dtype=DTYPES[dtype], device=DEV)
    at = 2 * G * D + H * V
    kernels.delta_rule(row[:, :G * D], row[:, G * D:2 * G * D], row[:, 2 * G * D:at], row[:, at:at + H], row[:, at + H:], dev(a_log), dev(dt_bias),
                       ctx, SimpleNamespace(buffer=bad, slots=ints([8])), o, H, G, D, V, status)
    assert int(status.item()) == 1 and (bad == 7.0).all()                      # a slot outside the buffer is flagged, not touched


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2, 5, 9), (3, 12, 4), (2, 16, 16), (2, 64, 40), (1, 130, 64), (4, 128, 128)])
def test_forget_and_write_whole_portions_and_single_tokens(sizes, dtype):
    """The forget gate with a floor: floors of 0 and near 1, gates from shut to open, long requests in chunks side by side."""
    from sprout_lm_b200 import kernels
    H, D, V = sizes
    rng = np.random.default_rng(H * 100 + D)
    lengths = dict(enumerate((300, 1, 129, 64, 5)))
    floor = rng.uniform(0.0, 0.95, H * D).astype(np.float32)
    floor[::3] = 0.0
    bias = np.linspace(-3.0, 8.0, H * D).astype(np.float32)
    data, want = {}, {}
    for r, n in lengths.items():
        data[r] = {key: rounded(v, dtype) for key, v in (("q", rng.normal(0, 2.0, size=(n, H * D))), ("z", rng.normal(0, 2.0, size=(n, H * D))),
                                                         ("v", rng.normal(size=(n, H * V))))}
        d = {key: f64(v) for key, v in data[r].items()}
        f = floor + (1.0 - floor.astype(np.float64)) * plain.sigmoid(d["z"] + bias)
        want[r] = plain.forget_and_write(plain.silu(d["q"]).reshape(n, H, D), f.reshape(n, H, D), d["v"].reshape(n, H, V))
    status = new_status()

    def stepper(state):
        def step(pieces, slots):
            ctx, slot_ids, counts = batch_context(pieces, slots)
            rows = dev(torch.cat([torch.cat([data[r][key][a:b] for key in ("q", "z", "v")], dim=1) for r, (a, b) in pieces.items()]), dtype)
            o = torch.empty(rows.shape[0], H * V, dtype=torch.float32, device=DEV)
            kernels.gated_scan(rows[:, :H * D], None, rows[:, 2 * H * D:], rows[:, H * D:2 * H * D], dev(bias), ctx,
                               SimpleNamespace(buffer=state, slots=slot_ids), o, H, H, D, V, status, floor=dev(floor), q_silu=True)
            return split(o.cpu().numpy().reshape(-1, H, V), pieces, counts)
        return step

    for label, cycle, slots in (("whole", (400,), {0: 4, 1: 0, 2: 5, 3: 2, 4: 1}), ("portions", (17, 2, 131, 1, 64, 3, 128), {0: 1, 1: 3, 2: 0, 3: 5, 4: 2}),
                                ("single", (1,), {0: 5, 1: 4, 2: 3, 3: 2, 4: 0})):
        state = torch.full((6, H, D, V), 7.0, dtype=torch.float32, device=DEV)
        for s in slots.values():
            state[s].zero_()
        got = drive(lengths, slots, cycle, stepper(state), limit=40 if label == "single" else None, holdout=label == "portions")
        for r, (o, S) in want.items():
            n = len(got[r])
            assert np.abs(got[r] - o[:n]).max() <= 5e-5 * max(1.0, np.abs(o).max()), (label, r, np.abs(got[r] - o[:n]).max())
            if n == len(o):
                assert np.abs(state[slots[r]].cpu().numpy() - S).max() <= 5e-5 * max(1.0, np.abs(S).max()), (label, r)
    assert int(status.item()) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("taps", [2, 3, 4, 6, 8])
def test_short_convolution_without_bias(taps, dtype):
    """Portions shorter than the taps, the first tokens of a sequence, other requests beside, with silu and without."""
    from sprout_lm_b200 import kernels
    rng = np.random.default_rng(taps)
    channels = 21
    lengths = dict(enumerate((70, 1, 9, 33)))
    weight = rng.normal(size=(channels, taps)).astype(np.float32)
    data = {r: rounded(rng.normal(size=(n, channels)), dtype) for r, n in lengths.items()}
    for silu in (False, True):
        for cycle in ((100,), (2, 1, 5, 34, 3), (1,)):
            slots = {0: 2, 1: 0, 2: 4, 3: 1}
            state = torch.full((5, taps - 1, channels), 7.0, dtype=torch.float32, device=DEV)
            for s in slots.values():
                state[s].zero_()
            status = new_status()

            def step(pieces, slots):
                ctx, slot_ids, counts = batch_context(pieces, slots)
                rows = dev(torch.cat([data[r][a:b] for r, (a, b) in pieces.items()]), dtype)
                out = torch.empty_like(rows)
                kernels.causal_conv(rows, dev(weight), None, out, ctx, SimpleNamespace(buffer=state, slots=slot_ids), status, silu=silu)
                return split(out.float().cpu().numpy(), pieces, counts)
            got = drive(lengths, slots, cycle, step)
            for r in lengths:
                want = plain.short_conv(f64(data[r]), weight.astype(np.float64))
                want = plain.silu(want) if silu else want
                assert (np.abs(got[r] - want) <= (1e-5 if dtype == "float32" else 1e-2) * (1 + np.abs(want))).all(), (r, silu, cycle)
            assert int(status.item()) == 0


# ------------------------------------------------------------------------------- attention
def _tables(kind, dims, base):
    from sprout_lm_b200.config.specs import PartSpec
    from sprout_lm_b200.parts import build_part
    if not dims:
        return None, None
    part = build_part("position", PartSpec(kind, {"dims": dims, "theta": base, "max_positions": 2048, "scaling": None}), "")
    return part.rotary_tables(SimpleNamespace(device=DEV))


# (heads, kv heads, dim, vdim, rotated, interleaved, page, window or None, turned values, unit-length vectors, whole-projection
#  norm, unit sink, gate)
ATTENTION_CASES = [
    (4, 2, 6, 10, 4, True, 16, 5, True, True, False, False, "head"),
    (3, 3, 8, 6, 8, False, 8, None, False, False, True, True, "element"),
    (2, 1, 12, 4, 12, True, 8, 9, True, True, False, False, "head"),
    (4, 4, 16, 16, 0, True, 16, 33, True, True, False, False, "head"),
    (2, 1, 10, 12, 6, False, 16, None, True, False, True, True, "element"),
    (8, 2, 64, 128, 32, True, 16, 100, True, True, False, False, "head"),
    (4, 1, 32, 64, 32, True, 16, 70, True, True, False, False, "head"),
    (2, 2, 96, 96, 64, False, 16, None, False, False, True, True, "element"),
    (4, 2, 64, 64, 64, False, 32, None, False, False, True, True, "element"),
    (4, 4, 48, 48, 48, False, 16, 130, True, False, True, True, "element"),
    (6, 3, 80, 80, 40, True, 8, 1, True, True, False, True, "head"),
    (8, 1, 128, 128, 128, False, 16, 64, True, True, False, False, "head"),
    (16, 1, 32, 32, 32, True, 16, None, True, True, False, True, "element"),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ATTENTION_CASES)
def test_attention_with_turned_values_norms_sinks_and_gates(dtype, case):
    """Norms, rotation, append and attention together, in contexts on both sides of page, window and 64-key borders; portions
    of queries and single queries (whose keys several CTAs divide); pages in shuffled order, unused pages not a number."""
    from sprout_lm_b200 import kernels
    H, G, dim, vdim, rot, inter, page, window, turned, unit, whole, unit_sink, gate_kind = case
    rng = np.random.default_rng(sum(int(x or 0) for x in case[:9]))
    base, eps, scale = 300.0, 1e-5, 1.4 / np.sqrt(dim) * (3.0 if not whole else 1.0)
    kind = "rope_interleaved" if inter else "rope_yarn"
    cos, sin = _tables(kind, rot, base)
    turn = _tables(kind, vdim, base) if turned else None
    mask = None if window is None else ("window", window)
    edges = sorted({1, 2, page, page + 1, 63, 64, 65, 127, 129, 200, 333} | ({window - 1, window, window + 1, 2 * window + 3} if window else set()))
    contexts = [n for n in edges if n >= 1][:14]
    q_lens = [min(n, q) for n, q in zip(contexts, (1, 1, 2, 1, 5, 1, 17, 1, 64, 1, 3, 1, 40, 1))]
    pages_per = [-(-n // page) for n in contexts]
    total = sum(pages_per) + 3
    order = rng.permutation(total)[:sum(pages_per)]
    table = np.full((len(contexts), max(pages_per)), -1, dtype=np.int32)
    at = 0
    for r, n in enumerate(pages_per):
        table[r, :n] = order[at:at + n]
        at += n
    k_cache = torch.full((total, G, page, dim), float("nan"), dtype=DTYPES[dtype], device=DEV)
    v_cache = torch.full((total, G, page, vdim), float("nan"), dtype=DTYPES[dtype], device=DEV)
    status = new_status()
    qw = rng.uniform(0.4, 1.8, size=H * dim).astype(np.float32) if whole else None
    kw = rng.uniform(0.4, 1.8, size=G * dim).astype(np.float32) if whole else None
    sink = torch.zeros(H, dtype=torch.float32, device=DEV) if unit_sink else None
    gate_width = H if gate_kind == "head" else H * vdim
    wants, q_rows, gate_rows, starts = [], [], [], [0]
    for r, (n, ql) in enumerate(zip(contexts, q_lens)):
        q, k, v = (rounded(rng.normal(size=(n, heads, d)), dtype) for heads, d in ((H, dim), (G, dim), (G, vdim)))
        gate = rounded(rng.normal(0, 2.0, size=(n, gate_width)), dtype)
        rows = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], dim=1)
        pad = -rows.shape[1] % 8
        rows = dev(torch.cat([rows, torch.zeros(n, pad)], dim=1), dtype)
        kernels.rope_maps_append(rows, ints(range(n)), ints([r] * n), dev(table), cos, sin, k_cache, v_cache, H, G, 1, dim, vdim, page, True,
                                 status, unit_eps=eps if unit else 0.0, q_weight=None if qw is None else dev(qw),
                                 k_weight=None if kw is None else dev(kw), weight_eps=eps, interleaved=inter, value_turn=turn)
        q_rows.append(rows[n - ql:, :H * dim])
        gate_rows.append(gate[n - ql:])
        starts.append(starts[-1] + ql)
        pq, pk, pv, pos = f64(q), f64(k), f64(v), np.arange(n)
        if whole:
            pq = plain.rms_norm(pq.reshape(n, -1), qw, eps).reshape(n, H, dim)
            pk = plain.rms_norm(pk.reshape(n, -1), kw, eps).reshape(n, G, dim)
        pq, pk = plain.rotate(pq, pos, base, rot, inter), plain.rotate(pk, pos, base, rot, inter)
        if unit:
            pq, pk = plain.unit_rms(pq, eps), plain.unit_rms(pk, eps)
        if turned:
            pv = plain.rotate(pv, pos, base, vdim, inter)
        o = plain.softmax_attention(pq, pk, pv, scale, window=window, unit_sink=unit_sink)
        if turned:
            o = plain.rotate(o, -pos, base, vdim, inter)
        g = plain.sigmoid(f64(gate))
        o = o * (g[:, :, None] if gate_kind == "head" else g.reshape(n, H, vdim)) * 0.7
        wants.append(o[n - ql:].reshape(ql, H * vdim))
    assert int(status.item()) == 0
    q_all, gates, want = torch.cat(q_rows), dev(torch.cat(gate_rows), dtype), np.concatenate(wants)
    positions = np.concatenate([np.arange(n - ql, n) for n, ql in zip(contexts, q_lens)])
    seq_of = np.concatenate([[r] * ql for r, ql in enumerate(q_lens)])
    tol = 3e-5 if dtype == "float32" else 6e-2       # 16 bits: queries, keys and values are rounded after norm and rotation

    def run(sel, max_q_len, planned):
        rows = np.concatenate([np.arange(starts[r], starts[r + 1]) for r in sel])
        ctx = SimpleNamespace(q_start=ints(np.concatenate([[0], np.cumsum([q_lens[r] for r in sel])])), positions=ints(positions[rows]),
                              seq_of_token=ints([sel.index(r) for r in seq_of[rows]]), max_q_len=max_q_len, planned_context=planned,
                              max_context=max(contexts))
        part = SimpleNamespace(k=k_cache, v=v_cache, block_table=dev(table)[torch.tensor(sel, device=DEV)].contiguous(),
                               page_tokens=page, write=False)
        wide = torch.zeros(len(rows), -(-H * dim // 8) * 8, dtype=DTYPES[dtype], device=DEV)
        wide[:, :H * dim] = q_all[rows]
        out = torch.empty(len(rows), H * vdim, dtype=DTYPES[dtype], device=DEV)
        kernels.multimap_attention(wide[:, :H * dim], part, ctx, out, H, G, 1, dim, vdim, scale, 0.0, 0.0, 0.7, status, mask=mask, sink=sink,
                                   gate=gates[rows].contiguous(), turn=turn, interleaved=inter)
        err = np.abs(out.float().cpu().numpy() - want[rows]).max()
        assert err <= tol, (sel, err)
    everyone = list(range(len(contexts)))
    run(everyone, max(q_lens), max(contexts))                               # portions beside single queries
    singles = [r for r in everyone if q_lens[r] == 1]
    run(singles, 1, max(contexts[r] for r in singles))                      # a step of single tokens, its keys divided among CTAs
    run(singles[-1:], 1, contexts[singles[-1]])
    assert int(status.item()) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_key_decides(dtype):
    """Where random numbers would hide a fault: one key's score stands out, far back among hundreds, just inside and just
    outside the window, in a prompt portion and in a single-token step; its value must come back turned by the distance alone
    to that key; and a context whose scores are all far below zero, where the added one takes nearly all the weight."""
    from sprout_lm_b200 import kernels
    H, G, dim, vdim, page, window, base = 4, 2, 64, 64, 16, 70, 5000.0
    rng = np.random.default_rng(9)
    n, status = 333, new_status()
    turn = _tables("rope_interleaved", vdim, base)
    table = rng.permutation(40)[:21].astype(np.int32).reshape(1, 21)
    for place, mask, seen in ((n - 1 - 69, ("window", window), True), (n - 1 - 70, ("window", window), False), (0, None, True), (3, None, True),
                              (n - 1, ("window", window), True), (0, ("window", n), True), (0, ("window", n - 1), False), (n - 64, None, True)):
        k, v, q = rng.normal(0, 0.05, size=(n, G, dim)), rng.normal(size=(n, G, vdim)), rng.normal(0, 0.05, size=(n, H, dim))
        direction = rng.normal(size=dim)
        direction /= np.linalg.norm(direction)
        k[place] = direction * 6.0
        q[n - 1] = direction * 6.0                                          # score 36 * scale at one key, near zero elsewhere
        q_t, k_t, v_t = rounded(q, dtype), rounded(k, dtype), rounded(v, dtype)
        k_cache = torch.zeros((40, G, page, dim), dtype=DTYPES[dtype], device=DEV)
        v_cache = torch.zeros((40, G, page, vdim), dtype=DTYPES[dtype], device=DEV)
        rows = dev(torch.cat([q_t.reshape(n, -1), k_t.reshape(n, -1), v_t.reshape(n, -1)], dim=1), dtype)
        kernels.rope_maps_append(rows, ints(range(n)), ints([0] * n), dev(table), None, None, k_cache, v_cache, H, G, 1, dim, vdim, page,
                                 True, status, interleaved=True, value_turn=turn)
        view = SimpleNamespace(k=k_cache, v=v_cache, block_table=dev(table), page_tokens=page, write=False)
        chosen = plain.rotate(f64(v_t)[place:place + 1], np.array([place - (n - 1)]), base, vdim, True)[0]         # [G, vdim]
        for q_len in (1, 23):
            ctx = SimpleNamespace(q_start=ints([0, q_len]), positions=ints(range(n - q_len, n)), seq_of_token=ints([0] * q_len),
                                  max_q_len=q_len, planned_context=n, max_context=n)
            out = torch.empty(q_len, H * vdim, dtype=DTYPES[dtype], device=DEV)
            kernels.multimap_attention(rows[n - q_len:, :H * dim], view, ctx, out, H, G, 1, dim, vdim, 0.5, 0.0, 0.0, 1.0, status,
                                       mask=mask, turn=turn, interleaved=True)
            last = out[-1].float().cpu().numpy().reshape(H, vdim)
            near = all(np.abs(last[h] - chosen[h // 2]).max() < 0.08 for h in range(H))
            assert near == seen, (place, mask, q_len)
    for shift, share in ((-40.0, 0.0), (40.0, 1.0)):
        # every score is shift (one query and keys that all agree): with one in the denominator the output vanishes or stays
        k_cache.zero_()
        k_cache[..., 0] = shift
        q_one = torch.zeros(1, H * dim, dtype=DTYPES[dtype], device=DEV)
        q_one[:, ::dim] = 1.0
        ctx = SimpleNamespace(q_start=ints([0, 1]), positions=ints([n - 1]), seq_of_token=ints([0]), max_q_len=1, planned_context=n,
                              max_context=n)
        out = torch.empty(1, H * vdim, dtype=DTYPES[dtype], device=DEV)
        kernels.multimap_attention(q_one, view, ctx, out, H, G, 1, dim, vdim, 1.0, 0.0, 0.0, 1.0, status,
                                   sink=torch.zeros(H, dtype=torch.float32, device=DEV))
        mean = v_cache[torch.from_numpy(table[0].astype(np.int64)).to(DEV)].float().permute(0, 2, 1, 3).reshape(-1, G, vdim)[:n].mean(dim=0)
        want = mean.repeat_interleave(H // G, dim=0).reshape(1, -1) * share
        assert (out.float() - want).abs().max().item() <= 2e-2
    assert int(status.item()) == 0


# ------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sigmoid_routing_and_experts_weighed_on_their_input(dtype):
    """The choice by single sigmoids (also where they all round to one), weights that are the scores, and experts whose input
    the weight multiplies: few tokens and many, sizes the tensor-core products take and sizes they do not."""
    from sprout_lm_b200 import kernels
    rng = np.random.default_rng(4)
    for width, experts, top, ff, tokens, level in ((36, 5, 2, 12, 5, 0.0), (64, 6, 1, 24, 300, 0.0), (128, 8, 2, 32, 70, 0.0),
                                                   (64, 16, 3, 64, 3, 0.0), (72, 40, 8, 40, 130, 0.0), (64, 8, 2, 16, 20, 30.0)):
        h = rounded(rng.normal(size=(tokens, width)), dtype)
        router = rng.normal(0, 0.4, size=(experts, width)).astype(np.float32)
        if level:
            h[:, 0] = 1.0
            router[:, 0] = level                                               # every sigmoid is one in 32 bits; the products still differ
        want_ids, want_w = plain.route(f64(h), router.astype(np.float64), top)
        ids = torch.empty((tokens, top), dtype=torch.int32, device=DEV)
        weights = torch.empty((tokens, top), dtype=torch.float32, device=DEV)
        counts = torch.zeros(experts, dtype=torch.int32, device=DEV)
        kernels.moe_route(dev(h, dtype), dev(router), None, ids, weights, counts, experts, top, 1.0, renormalize=False, sigmoid=True)
        assert np.array_equal(ids.cpu().numpy(), want_ids), (width, experts)
        assert np.abs(weights.cpu().numpy() - want_w).max() <= 2e-6
        w = {"m.router": router.astype(np.float64)}
        gate, up, down = (rounded(rng.normal(0, 0.4, size=(experts, *shape)), dtype) for shape in ((ff, width), (ff, width), (width, ff)))
        for e in range(experts):
            w |= {f"m.e{e}.gate": f64(gate[e]), f"m.e{e}.up": f64(up[e]), f"m.e{e}.down": f64(down[e])}
        offsets = torch.zeros(experts + 1, dtype=torch.int32, device=DEV)
        order, place_of = (torch.empty(tokens * top, dtype=torch.int32, device=DEV) for _ in range(2))
        kernels.moe_arrange(ids, counts, offsets, order, place_of, experts)
        act = torch.empty((tokens * top, ff), dtype=DTYPES[dtype], device=DEV)
        rows = torch.empty((tokens * top, width), dtype=torch.float32, device=DEV)
        kernels.moe_experts(dev(h, dtype), order, offsets, dev(torch.cat([gate, up], dim=1), dtype), dev(down, dtype), act, rows, experts, top,
                            0.0, 0.0, unit="silu_glu", row_weights=weights)
        y = torch.ones((tokens, width), dtype=torch.float32, device=DEV)
        kernels.moe_combine(y, dev(h, dtype), ids, None, place_of, rows, top, factor=0.4)
        want = 1.0 + 0.4 * plain.moe_mlp(f64(h), w, "m.", {"router": {"experts": experts, "top": top}})
        err = np.abs(y.cpu().numpy() - want).max()
        assert err <= (3e-5 if dtype == "float32" else 3e-2) * max(1.0, np.abs(want).max()), (width, experts, tokens, err)


# =============================================================================== whole models
@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    base = tmp_path_factory.mktemp("zevedra")
    return {name: zh.make_model_dir(base, name) for name in zh.CONFIGS}


def make_requests(name, seed, lengths):
    vocab = zh.CONFIGS[name][0]["vocab"]
    rng = np.random.default_rng(seed)
    return {f"r{i}": helpers.random_tokens(rng, n, vocab) for i, n in enumerate(lengths)}


def make_runner(model_dir, dtype, pages, page_tokens, requests=4):
    from sprout_lm_b200.engine.step import ModelRunner
    from sprout_lm_b200.models import load_model
    model = load_model(model_dir, dtype=DTYPES[dtype])
    return ModelRunner(model, num_pages=pages, page_tokens=page_tokens, max_requests=requests, prefix_caching=False)


def test_layers_one_by_one(model_dirs):
    """The stream after every layer run in 32-bit (a looped layer counts each time), so that a fault names its layer."""
    from sprout_lm_b200.engine.batch import StepEntry
    for name, directory in model_dirs.items():
        config, tensors = zh.plain_model(directory)
        tokens = make_requests(name, 1, [41])["r0"]
        runner = make_runner(directory, "float32", 8, zh.CONFIGS[name][2])
        seen = []
        for block in runner.model.blocks:
            def wrapped(x, *args, _inner=block.forward, **more):
                _inner(x, *args, **more)
                seen.append(x.clone())
            block.forward = wrapped
        seq = runner.new_sequence()
        assert runner.reserve(seq, len(tokens))
        runner.step([StepEntry(seq, tokens, [0])])
        _, want = plain.forward(config, tensors, tokens, return_layers=True)
        assert len(seen) == len(want) == len(plain.run_order(config))
        for i, (got, expected) in enumerate(zip(seen, want)):
            assert np.abs(got.cpu().numpy() - expected).max() <= 3e-5 * max(1.0, np.abs(expected).max()), (name, "layer run", i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_all_cuttings_in_process(model_dirs, name, dtype):
    """Whole, tail decoded token by token (110 tokens: every window of the models passes over decoded tokens), portions
    down to two tokens, mixed batches with pages and state slots used again: against the plain implementation, and in 32-bit
    equal to one another to rounding."""
    page = zh.CONFIGS[name][2]
    requests = make_requests(name, 11, [5, 17, 33, 70, 150, 1, 40])
    rng = np.random.default_rng(5)
    plans = {
        "whole": helpers.plan_whole(requests),
        "tail": helpers.plan_tail_decode(requests, tail=110),
        "portions": helpers.plan_portions(requests),
        "mixed": helpers.plan_mixed(requests, rng),
    }
    results = {}
    for label, plan in plans.items():
        budget = helpers.live_token_budget(plan, requests)
        runner = make_runner(model_dirs[name], dtype, budget // page, page, requests=4)
        got = results[label] = helpers.run_plan_in_process(runner, plan)
        assert len(got) == sum(len(t) for t in requests.values())
        worst = zh.compare(model_dirs[name], requests, got, TOL[dtype], f"{name}/{dtype}/{label}", page, rounded=dtype == "bfloat16")
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
            zh.compare(model_dirs[name], requests, got, TOL[dtype], f"long/{name}/{dtype}", page, rounded=dtype == "bfloat16")


def test_trace_replay_program(model_dirs, tmp_path):
    """bin/trace_run picks the model class by config.json and replays a mixed plan with four state slots."""
    name = "B"
    requests = make_requests(name, 13, [9, 40, 70, 23, 31, 12])
    plan = helpers.plan_mixed(requests, np.random.default_rng(2))
    budget = helpers.live_token_budget(plan, requests)
    vocab = zh.CONFIGS[name][0]["vocab"]
    for dtype in ("float32", "bfloat16"):
        got = helpers.run_plan_with_trace_run(model_dirs[name], dtype, plan, tmp_path / dtype, budget, vocab=vocab)
        zh.compare(model_dirs[name], requests, got, TOL[dtype], f"trace/{dtype}", 16, rounded=dtype == "bfloat16")


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_scheduler(model_dirs, name):
    """generate(): continuous batching, chunked prefill and captured decode steps; in 32-bit the tokens are the plain
    implementation's, in bfloat16 every token is within bfloat16's reach of the plain choice."""
    from sprout_lm_b200 import generate, load_model
    config, tensors = zh.plain_model(model_dirs[name])
    rng = np.random.default_rng(7)
    prompts = [helpers.random_tokens(rng, n, config["vocab"]) for n in (3, 19, 44)]
    new_tokens = 12
    for dtype in ("float32", "bfloat16"):
        model = load_model(model_dirs[name], dtype=dtype)
        results = generate(model, prompts, max_new_tokens=new_tokens, ignore_eos=True)
        for prompt, result in zip(prompts, results):
            assert len(result["output"]) == new_tokens
            history = list(prompt)
            for token in result["output"]:
                row = plain.forward(config, tensors, history)[-1]
                spread = float(np.sqrt(np.mean((row - row.mean()) ** 2)))
                assert row[token] >= row.max() - (1e-4 if dtype == "float32" else 4 * TOL["bfloat16"]) * spread, (name, dtype, len(history))
                history.append(token)


def test_device_side_decode_loop(model_dirs):
    """Decode steps that run back to back on the device: the previous token a step's embedding needs is the one the device
    sampled the step before."""
    from sprout_lm_b200.engine.batch import StepEntry
    name = "A"
    directory, page = model_dirs[name], zh.CONFIGS[name][2]
    config, _ = zh.plain_model(directory)
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
        want = zh.plain_greedy(directory, prompt, len(history) + 1)
        assert [first[i], *history[:, i].tolist()] == want


def test_scheduler_under_page_pressure(model_dirs):
    """A pool smaller than the requests together: a preempted request gives its state slot back and recomputes its state
    from the start; the greedy tokens stay the plain implementation's."""
    from sprout_lm_b200 import EngineOptions, generate, load_model
    name = "A"
    config, _ = zh.plain_model(model_dirs[name])
    rng = np.random.default_rng(8)
    prompts = [helpers.random_tokens(rng, n, config["vocab"]) for n in (30, 41, 26, 35)]
    model = load_model(model_dirs[name], dtype="float32")
    options = EngineOptions(block_size=8, num_blocks=14, max_sequences=4, max_batch_tokens=24, prefill_chunk_size=7)
    results = generate(model, prompts, max_new_tokens=10, ignore_eos=True, options=options)
    for prompt, result in zip(prompts, results):
        assert result["output"] == zh.plain_greedy(model_dirs[name], prompt, 10)
