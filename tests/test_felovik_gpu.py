"""Felovik on the GPU against the plain float64 implementation (``tests/plain/felovik_plain.py``): each mechanism's kernels
alone, then whole models under every way of cutting and batching their requests, through the engine's own step function,
cache manager, scheduler and entry point. Sizes are the tests' own (``felovik_util.CONFIGS``)."""
import math

import numpy as np
import pytest
import torch

import conftest
from plain import felovik_plain as plain
import felovik_util as fu
import zurerax_util as zu

pytestmark = pytest.mark.gpu
DEV = "cuda:0"

# bfloat16 against float64: where two router scores lie closer than the rounding of the router's input, bfloat16 picks another
# expert than float64 and that token's logits differ by a discrete amount that the state carries on. So the bound holds for
# nine rows in ten and for the median row. Faults in which key, token or expert a bfloat16 kernel reads are caught by the
# crafted tests below and by the float32 runs of the same code, which are held to 1e-4.
BF16_REL_MAX, BF16_REL_MEAN, BF16_ROWS_OFF = 0.3, 0.04, 0.1


def assert_logits_close(got, want, dtype, what=""):
    if dtype == "float32":
        return conftest.assert_logits_close(got, want, dtype, what)
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all(), what
    diff, spread = np.abs(got - want), want.std()
    off = diff.max(1) > BF16_REL_MAX * spread
    assert off.sum() <= max(1, BF16_ROWS_OFF * len(off)), \
        f"{what}: {int(off.sum())} of {len(off)} rows differ by more than {BF16_REL_MAX} x spread {spread:.3e} (worst {diff.max():.3e})"
    assert np.median(diff.mean(1)) <= BF16_REL_MEAN * spread, \
        f"{what}: the median row's mean abs diff {np.median(diff.mean(1)):.3e} > {BF16_REL_MEAN} x spread {spread:.3e}"


def _i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def _f32(a):
    return torch.tensor(np.asarray(a, dtype=np.float32), device=DEV)


def _status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def _rounded(a, dtype):
    """``a`` as float64, rounded to ``dtype`` first, so that kernel and plain implementation start from the same numbers."""
    return torch.tensor(np.asarray(a), dtype=torch.float32).to(dtype).double().numpy()


def _step_meta(step, at):
    """Device metadata of one step of (request, rows) entries (None: a padding sequence of one row)."""
    row_seq, positions, first, start, row = [], [], [], [], 0
    for s, e in enumerate(step):
        first.append(row)
        if e is None:
            start.append(-1); row_seq.append(s); positions.append(-1); row += 1
            continue
        start.append(at[e[0]])
        row_seq += [s] * e[1]
        positions += [at[e[0]] + i for i in range(e[1])]
        row += e[1]
    first.append(row)
    return row, _i32(row_seq), _i32(positions), _i32(first), _i32(start)


def _cuts(lengths, rng, tail=True):
    """Steps that bring every request in: portions of changing sizes side by side (down to one and two rows), then (``tail``)
    the last third of each request token by token, all requests in one step, finished ones as padding sequences."""
    at, steps = [0] * len(lengths), []
    stop = [n - (n // 3 if tail else 0) for n in lengths]
    while any(a < s for a, s in zip(at, stop)):
        step = []
        for r in range(len(lengths)):
            if at[r] < stop[r] and rng.random() < 0.8:
                k = min(int(rng.choice([1, 2, 3, 15, 16, 17, 40, 63, 64, 65, 130])), stop[r] - at[r])
                step.append((r, k))
                at[r] += k
        if step:
            step.insert(int(rng.integers(0, len(step) + 1)), None)
            steps.append(step)
    while any(a < n for a, n in zip(at, lengths)):
        steps.append([(r, 1) if at[r] < lengths[r] else None for r in range(len(lengths))])
        for r in range(len(lengths)):
            at[r] += at[r] < lengths[r]
    return steps


def _gather(step, at, rows_in, width):
    n = sum(1 if e is None else e[1] for e in step)
    x, row = np.full((n, width), 99.0), 0                # (padding rows: a number that would show)
    for e in step:
        if e is None:
            row += 1
            continue
        x[row:row + e[1]] = rows_in[e[0]][at[e[0]]:at[e[0]] + e[1]]
        row += e[1]
    return x


def _scatter(step, at, out, got):
    row = 0
    for e in step:
        if e is None:
            row += 1
            continue
        got[e[0]][at[e[0]]:at[e[0]] + e[1]] = out[row:row + e[1]]
        row += e[1]
        at[e[0]] += e[1]


# ---------------------------------------------------------------------------------------------- each mechanism alone
def test_scaled_embedding_with_a_position():
    from glassbox_b200 import kernels
    rng = np.random.default_rng(0)
    W = {"embed": _rounded(rng.standard_normal((20, 37)), torch.bfloat16), "pos": _rounded(rng.standard_normal((9, 37)), torch.bfloat16)}
    tokens = [3, 19, 0, 3, 7]
    x = torch.full((6, 37), 5.0, device=DEV)
    kernels.embed_positions(_f32(W["embed"]).bfloat16(), _f32(W["pos"]).bfloat16(), _i32(tokens + [0]), _i32([0, 1, 2, 3, 4, -1]), x, _status(),
                            scale=2.7)
    np.testing.assert_allclose(x[:5].cpu().numpy(), plain.embed(W, tokens, 2.7), atol=1e-5, rtol=1e-6)
    assert not x[5].any()


@pytest.mark.parametrize("n, d", [(1, 50), (3, 257), (70, 128), (5, 2304), (2, 4096), (3, 5000)])
def test_norm_after_the_sum(n, d):
    """x <- w (alpha x + y) / rms(alpha x + y), y stored, as a weighted sum of rows, or as a pair of normed rows; a copy in the
    activation dtype; padding rows stay as they are."""
    from glassbox_b200 import kernels
    rng = np.random.default_rng(n * d)
    x, w = rng.standard_normal((n, d)), 1 + 0.2 * rng.standard_normal(d)
    a, b = rng.standard_normal((n, d)) * 3, rng.standard_normal((n, d)) * 0.2
    ga, gb = 1 + 0.3 * rng.standard_normal(d), 1 + 0.3 * rng.standard_normal(d)
    pair, weight, shared, gate = rng.standard_normal((n, 3, d)), rng.random((n, 3)), rng.standard_normal((n, d)), rng.random(n)
    positions = [4] * n
    if n > 2:
        positions[1] = -1
    live = np.array(positions) >= 0
    pair_dev = _f32(pair.reshape(n, 3 * d))
    cases = [(_f32(a), a), (kernels.WeightedRows(pair_dev, _f32(weight)), (weight[..., None] * pair).sum(1)),
             (kernels.WeightedRows(pair_dev, _f32(weight), _f32(shared), _f32(gate)), (weight[..., None] * pair).sum(1) + gate[:, None] * shared),
             (kernels.NormedPair(_f32(a), _f32(b), _f32(ga), _f32(gb), 0.5, 0.25, 1e-5),
              0.5 * plain.rms_unit(a, 1e-5) * ga + 0.25 * plain.rms_unit(b, 1e-5) * gb)]
    for branch, y in cases:
        for copy_dtype in (None, torch.bfloat16, torch.float32):
            xs = _f32(x)
            copy = torch.zeros((n, d), dtype=copy_dtype, device=DEV) if copy_dtype else None
            kernels.post_norm(xs, _f32(w), 1.7, 1e-6, branch, positions=_i32(positions), copy=copy)
            want = plain.rms_unit(1.7 * x + y, 1e-6) * w
            np.testing.assert_allclose(xs.cpu().numpy()[live], want[live], atol=3e-5, rtol=1e-5)
            np.testing.assert_array_equal(xs.cpu().numpy()[~live], x.astype(np.float32)[~live])
            if copy is not None:
                assert torch.equal(copy[torch.tensor(live)], xs[torch.tensor(live)].to(copy_dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n, groups, size", [(1, 1, 1), (5, 3, 7), (9, 8, 16), (4, 2, 300), (3, 1, 2048), (2, 1, 5000)])
def test_gate_then_norm_in_parts(dtype, n, groups, size):
    from glassbox_b200 import kernels
    rng = np.random.default_rng(size)
    w = groups * size
    y, z, g = rng.standard_normal((n, w)) * 2, rng.standard_normal((n, w + 3)) * 2, rng.standard_normal(w)
    for off in (0, 3):                                   # (a column slice that starts 16-byte aligned, and one that does not)
        out = torch.zeros((n, w), dtype=dtype, device=DEV)
        kernels.gate_group_norm(_f32(y), _f32(z)[:, off:off + w], _f32(g), out, groups, 1e-5)
        want = plain.grouped_gated_norm(y, z[:, off:off + w], g, groups, 1e-5)
        np.testing.assert_allclose(out.float().cpu().numpy(), want, atol=2e-5 if dtype == torch.float32 else 3e-2, rtol=1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("C, taps, col", [(24, 4, 0), (40, 1, 4), (64, 2, 0), (512, 3, 8), (37, 4, 0), (16, 5, 3), (12, 7, 0)])
def test_convolution_over_a_ring(C, taps, col):
    """Every portion continues from the ring of the request's last inputs, wherever it was cut; foreign slots are left alone,
    padding rows too; both output dtypes."""
    from glassbox_b200 import kernels
    rng = np.random.default_rng(C + taps)
    lengths = [150, 7, 41]
    rows_in = [rng.standard_normal((n, C)) for n in lengths]
    w, b = rng.standard_normal((C, taps)) * 0.6, rng.standard_normal(C)
    off, slots = 8, [3, 0, 5]
    state = torch.zeros((7, off + taps * C + 4), device=DEV)
    state[:, :off], state[[1, 2, 4, 6]] = 7.0, 7.0
    got = [np.zeros((n, C)) for n in lengths]
    at = [0, 0, 0]
    for step in _cuts(lengths, rng):
        n, row_seq, positions, first, start = _step_meta(step, at)
        x = torch.full((n, C + col + 5), 50.0, device=DEV)
        x[:, col:col + C] = _f32(_gather(step, at, rows_in, C))
        y = torch.full((n, C), -3.0, device=DEV)
        status = _status()
        args = (row_seq, positions, first, start, _i32([6 if e is None else slots[e[0]] for e in step]))
        before = state.clone()
        half = torch.zeros((n, C), dtype=torch.bfloat16, device=DEV)
        kernels.ring_conv(x[:, col:col + C], _f32(w), _f32(b), half, state, off, *args, False, status)
        assert torch.equal(state, before)
        kernels.ring_conv(x[:, col:col + C], _f32(w), _f32(b), y, state, off, *args, True, status)
        assert int(status.item()) == 0
        live = positions >= 0
        np.testing.assert_allclose(half[live].float().cpu().numpy(), y[live].cpu().numpy(), atol=2e-2, rtol=1e-2)
        _scatter(step, at, y.cpu().numpy(), got)
    for r, rows in enumerate(rows_in):
        np.testing.assert_allclose(got[r], plain.silu(plain.causal_conv(rows, w, b)), atol=2e-5, rtol=1e-5)
    ring = state[:, off:off + taps * C].view(7, taps, C).cpu().numpy()
    for r, n in enumerate(lengths):
        for p in range(max(0, n - taps), n):
            np.testing.assert_array_equal(ring[slots[r], p % taps], rows_in[r][p].astype(np.float32))
    assert bool((state[[1, 2, 4, 6]] == 7.0).all()) and bool((state[:, :off] == 7.0).all())


def test_convolution_leaves_the_rows_and_requests_before_its_share_alone():
    from glassbox_b200 import kernels
    rng = np.random.default_rng(3)
    step, at = [(0, 1), (1, 1), (2, 9)], [4, 0, 0]
    n, row_seq, positions, first, start = _step_meta(step, at)
    x, w, b = rng.standard_normal((n, 16)), rng.standard_normal((16, 3)), rng.standard_normal(16)
    state = torch.full((3, 48), 2.0, device=DEV)
    y = torch.full((n, 16), -3.0, device=DEV)
    kernels.ring_conv(_f32(x), _f32(w), _f32(b), y, state, 0, row_seq, positions, first, start, _i32([0, 1, 2]), True, _status(),
                      first_row=2, first_seq=2)
    assert bool((y[:2] == -3.0).all()) and bool((state[:2] == 2.0).all())
    np.testing.assert_allclose(y[2:].cpu().numpy(), plain.silu(plain.causal_conv(x[2:], w, b)), atol=2e-5)


def _ssd_inputs(rng, lengths, H, G, N, V, dtype):
    inner, gn = H * V, G * N
    rows = [_rounded(rng.standard_normal((n, inner + 2 * gn)), dtype) for n in lengths]
    dts = [rng.standard_normal((n, H)) * 1.5 - 1.0 for n in lengths]
    params = {"dt_bias": rng.standard_normal(H), "a_log": rng.uniform(-3.0, 2.0, H), "skip": rng.standard_normal(H)}
    return rows, dts, params


def _ssd_want(rows, dts, p, H, G, N, V):
    inner, gn, out = H * V, G * N, []
    for x, dt in zip(rows, dts):
        T = len(x)
        y = plain.ssd_scan(x[:, :inner].reshape(T, H, V), x[:, inner:inner + gn].reshape(T, G, N), x[:, inner + gn:].reshape(T, G, N),
                           plain.softplus(dt + p["dt_bias"]), p["a_log"], p["skip"])
        out.append(y.reshape(T, inner))
    return out


def _run_ssd(how, steps, rows, dts, p, H, G, N, V, slots, state):
    from glassbox_b200 import kernels
    C = H * V + 2 * G * N
    dtype = torch.bfloat16 if how == "chunks" else torch.float32
    got = [np.zeros((len(r), H * V)) for r in rows]
    at = [0] * len(rows)
    p = {k: _f32(v) for k, v in p.items()}
    for step in steps:
        n, row_seq, positions, first, start = _step_meta(step, at)
        x, dt = _f32(_gather(step, at, rows, C)).to(dtype), _f32(_gather(step, at, dts, H))
        y = torch.full((n, H * V), -3.0, device=DEV)
        status = _status()
        meta = (first, start, _i32([len(state) - 1 if e is None else slots[e[0]] for e in step]))
        args = (x, dt, p["dt_bias"], p["a_log"], p["skip"], state, y, *meta)
        if how == "chunks":
            need = kernels.ssd_chunks_needed(n, len(step))
            own = torch.full((need, H * N * V), float("nan"), device=DEV)
            steps = torch.full((need, H * 2 * kernels.ssd_chunk_rows()), float("nan"), device=DEV)
            kernels.ssd_chunks(*args, max(e[1] for e in step if e), H, G, N, V, True, status, own, steps)
        else:
            kernels.ssd_walk(*args, H, G, N, V, True, status)
        assert int(status.item()) == 0
        _scatter(step, at, y.cpu().numpy(), got)
    return got


@pytest.mark.parametrize("how", ["walk", "chunks"])
@pytest.mark.parametrize("H, G, N, V", [(4, 2, 16, 32), (2, 1, 128, 64), (3, 3, 24, 8), (6, 2, 10, 7), (1, 1, 1, 1), (2, 2, 40, 96)])
def test_the_recurrence_over_portions(how, H, G, N, V):
    """Portions cut anywhere, several requests a step, padding sequences between them, states carried from step to step; the
    final state of every slot and the foreign slots. Step logits and rates reach from hardly any decay to almost all."""
    rng = np.random.default_rng(N + V)
    lengths = [200, 5, 131]
    rows, dts, p = _ssd_inputs(rng, lengths, H, G, N, V, torch.bfloat16)
    state = torch.zeros((6, H * N * V + 12), device=DEV)
    state[[1, 4, 5]] = 3.0
    slots = [2, 0, 3]
    got = _run_ssd(how, _cuts(lengths, rng), rows, dts, p, H, G, N, V, slots, state)
    want = _ssd_want(rows, dts, p, H, G, N, V)
    for r in range(3):
        scale = np.abs(want[r]).max()
        np.testing.assert_allclose(got[r] / scale, want[r] / scale, atol=3e-5 if how == "chunks" else 2e-6)
    assert bool((state[[1, 4, 5]] == 3.0).all()) and not state[[0, 2, 3], H * N * V:].any()
    # the state of the longest request, from the equations
    g = [h // (H // G) for h in range(H)]
    dt = plain.softplus(dts[0] + p["dt_bias"])
    for h in range(H):
        S = np.zeros((N, V))
        for t in range(lengths[0]):
            B = rows[0][t, H * V + g[h] * N:H * V + (g[h] + 1) * N]
            S = math.exp(-math.exp(p["a_log"][h]) * dt[t, h]) * S + dt[t, h] * np.outer(B, rows[0][t, h * V:(h + 1) * V])
        top = np.abs(S).max()
        np.testing.assert_allclose(state[2, h * N * V:(h + 1) * N * V].view(N, V).cpu().numpy() / top, S / top, atol=3e-5)


@pytest.mark.parametrize("how", ["walk", "chunks"])
def test_the_recurrence_remembers_one_token(how):
    """With no decay and one value that is not zero, a read-out is that value from its own token on and zero before: at the
    first tokens, around the edges of chunks and of portions, and far behind."""
    H, G, N, V, T = 2, 1, 16, 8, 330
    one = math.log(math.e - 1.0)                          # softplus of it is 1
    p = {"dt_bias": np.full(H, one), "a_log": np.full(H, -60.0), "skip": np.zeros(H)}
    for mark in (0, 1, 62, 63, 64, 65, 127, 128, 200):
        x = np.zeros((T, H * V + 2 * G * N))
        x[:, H * V] = x[:, H * V + N] = 1.0               # B and C: the first state channel
        x[mark, :H * V] = 100.0
        for cuts in ([T], [64, 64, T - 128], [63, 2, 65, 1, T - 131], [mark + 1, T - mark - 1]):
            state = torch.zeros((1, H * N * V), device=DEV)
            got = _run_ssd(how, [[(0, k)] for k in cuts if k], [x], [np.zeros((T, H))], p, H, G, N, V, [0], state)[0]
            np.testing.assert_allclose(got[:mark], 0.0, atol=1e-3)
            np.testing.assert_allclose(got[mark:], 100.0, rtol=1e-5)


@pytest.mark.parametrize("H, G, N, V, taps", [(4, 2, 16, 32, 4), (2, 1, 128, 64, 3), (3, 3, 24, 8, 2), (6, 2, 10, 7, 4), (1, 1, 1, 1, 1),
                                             (2, 2, 40, 260, 5), (64, 8, 128, 64, 4)])
def test_single_tokens_in_one_kernel(H, G, N, V, taps):
    """Convolution over the ring, step, decay, update and read-out for unequal requests token by token, finished ones as
    padding sequences; the first tokens (an empty ring), foreign slots, and a pass that must not write."""
    from glassbox_b200 import kernels
    rng = np.random.default_rng(N * V + taps)
    lengths = [19, 3, 11] if H < 64 else [5, 2, 4]
    C = H * V + 2 * G * N
    raw = [rng.standard_normal((n, C)) for n in lengths]
    _, dts, p = _ssd_inputs(rng, lengths, H, G, N, V, torch.float32)
    w, b = rng.standard_normal((C, taps)) * 0.6, rng.standard_normal(C) * 0.3
    off = H * N * V + 4
    state = torch.zeros((5, off + taps * C), device=DEV)
    state[[1, 4]] = 3.0
    slots = [3, 0, 2]
    dev = {k: _f32(v) for k, v in p.items()}
    got = [np.zeros((n, H * V)) for n in lengths]
    at = [0] * 3
    for t in range(max(lengths)):
        step = [(r, 1) if t < lengths[r] else None for r in range(3)]
        n, _, _, first, start = _step_meta(step, at)
        x, dt = _f32(_gather(step, at, raw, C)), _f32(_gather(step, at, dts, H))
        meta = (first, start, _i32([4 if e is None else slots[e[0]] for e in step]))
        before, status = state.clone(), _status()
        ys = []
        for write in (False, True):
            y = torch.full((n, H * V), -3.0, device=DEV)
            kernels.ssd_decode(x, dt, _f32(w), _f32(b), dev["dt_bias"], dev["a_log"], dev["skip"], state, off, y, *meta, H, G, N, V, write, status)
            ys.append(y)
            if not write:
                assert torch.equal(state, before)
        assert torch.equal(ys[0], ys[1]) and int(status.item()) == 0
        _scatter(step, at, ys[1].cpu().numpy(), got)
    want = _ssd_want([plain.silu(plain.causal_conv(x, w, b)) for x in raw], dts, p, H, G, N, V)
    for r in range(3):
        np.testing.assert_allclose(got[r], want[r], atol=3e-5 * max(1.0, np.abs(want[r]).max()), rtol=1e-5)
    assert bool((state[[1, 4]] == 3.0).all())


class _Pages:
    """A paged cache for a few requests whose pages lie scattered and interleaved in the pool."""

    def __init__(self, lengths, G, D, V, page, dtype, seed=0):
        rng = np.random.default_rng(seed)
        need = [-(-n // page) for n in lengths]
        order = rng.permutation(sum(need) + 3)
        self.page, self.tables, at = page, [], 0
        for k in need:
            self.tables.append([int(p) for p in order[at:at + k]])
            at += k
        self.width = max(need)
        self.k = torch.zeros((sum(need) + 3, G, page, D), dtype=dtype, device=DEV)
        self.v = torch.zeros((sum(need) + 3, G, page, V), dtype=dtype, device=DEV)

    def row(self, seq):
        return self.tables[seq] + [-1] * (self.width - len(self.tables[seq]))

    def slot(self, seq, pos):
        return self.tables[seq][pos // self.page] * self.page + pos % self.page


def _by_identity(H, G, D, V):
    """Projections that pick a stacked row [q | k | v | gate] apart, and no output projection."""
    cols = (H + G) * D + G * V + H * V
    eye = np.eye(cols)
    return {"q": eye[:H * D], "k": eye[H * D:(H + G) * D], "v": eye[(H + G) * D:(H + G) * D + G * V], "g": eye[(H + G) * D + G * V:],
            "o": np.eye(H * V)}


def _run_attention(how, steps, rows_in, m, cache, dtype, eps):
    """Norm, temperature and cache write, then attention with its gate, step by step. ``how``: "rows", "decode" and "split" (the
    two kernels for single tokens; portions take the row kernel), "tiles" or "flash"."""
    from glassbox_b200 import kernels
    H, G, D, V, page = m["heads"], m["kv_heads"], m["dim"], m["vdim"], cache.page
    gate_col = (H + G) * D + G * V
    q_temp = (m["q_temp"]["coef"], m["q_temp"]["every"]) if m.get("q_temp") else None
    status = _status()
    got = [np.zeros((len(r), H * V)) for r in rows_in]
    at = [0] * len(rows_in)
    common = dict(r1=None, r2=None, sink=None, heads=H, kv_heads=G, dim=D, vdim=V, page_size=page, scale=m["scale"], window=None, status=status)
    for step in steps:
        n, row_seq, positions, first, start = _step_meta(step, at)
        proj = _f32(_gather(step, at, rows_in, gate_col + H * V))
        slots = [s for e in step for s in ([-1] if e is None else [cache.slot(e[0], at[e[0]] + i) for i in range(e[1])])]
        q, out = torch.zeros((n, H * D), dtype=dtype, device=DEV), torch.zeros((n, H * V), dtype=dtype, device=DEV)
        kernels.qk_norm_rope_write(proj[:, :gate_col], None, None, None, positions, _i32(slots), q, cache.k, cache.v, H, G, D, V, 0, eps, page,
                                   True, status, unit_norm=True, q_temp=q_temp)
        tables = _i32([[-1] * cache.width if e is None else cache.row(e[0]) for e in step])
        gate = proj[:, gate_col:]
        single = all(e is None or e[1] == 1 for e in step)
        longest = max(e[1] for e in step if e)
        if how == "flash":
            kernels.attention_prefill_tc(q, out, cache.k, cache.v, tables, first, start, longest, H, G, D, page, m["scale"], None, status,
                                         sink_terms=(None, None, None, gate))
        elif how == "tiles":
            kernels.sink_attention_tiles(q, out, cache.k, cache.v, tables, first, start, longest, gate=gate, **common)
        elif how == "split" and single:
            plans = [(1, 0, 4), (3, 16, 4), (2, 16, 8), (2, 0, 8), (5, 0, 4)] if D == 64 else [(1, 0, 4), (3, 0, 4), (2, 0, 4)]
            splits, block_keys, warps = plans[sum(at) % len(plans)]
            part_acc = torch.full((n, H * warps * splits * D), float("nan"), device=DEV)
            part_ml = torch.full((n, H * warps * splits * 2), float("nan"), device=DEV)
            counters = torch.zeros(n * G, dtype=torch.int32, device=DEV)
            kernels.attention_decode_mma(q, out, cache.k, cache.v, tables, row_seq, positions, H, G, D, page, m["scale"], None, splits, part_acc,
                                         part_ml, counters, status, block_keys, warps, sink_terms=(None, None, None, gate))
        elif how == "decode" and single:
            kernels.sink_attention_decode(q, out, cache.k, cache.v, tables, row_seq, positions, gate=gate, **common)
        else:
            kernels.sink_attention_rows(q, out, cache.k, cache.v, tables, row_seq, positions, gate=gate, **common)
        _scatter(step, at, out.float().cpu().numpy(), got)
    assert int(status.item()) == 0
    return got


ATTENTION_CASES = [("rows", "float32", 6, 2, 20, 12), ("rows", "float32", 3, 1, 9, 7), ("decode", "float32", 4, 2, 16, 32), ("decode", "bfloat16", 8, 2, 48, 64),
                   ("split", "bfloat16", 8, 2, 64, 64), ("split", "bfloat16", 4, 4, 32, 32), ("split", "bfloat16", 4, 1, 16, 16), ("split", "bfloat16", 4, 2, 128, 128),
                   ("tiles", "bfloat16", 4, 2, 64, 32),
                   ("tiles", "bfloat16", 6, 3, 48, 48), ("tiles", "bfloat16", 2, 1, 80, 80), ("tiles", "bfloat16", 2, 2, 96, 96),
                   ("flash", "bfloat16", 4, 2, 64, 64)]


@pytest.mark.parametrize("how, dtype, H, G, D, V", ATTENTION_CASES)
def test_attention_in_portions_over_scattered_pages(how, dtype, H, G, D, V):
    rng = np.random.default_rng(H * D + V)
    dt = getattr(torch, dtype)
    m = fu.left(H, G, D, V, (0.5, 9), scale=0.35)
    lengths = [150, 21, 67]
    rows_in = [rng.standard_normal((n, (H + G) * D + G * V + H * V)) for n in lengths]
    cache = _Pages(lengths, G, D, V, 16, dt)
    got = _run_attention(how, _cuts(lengths, rng), rows_in, m, cache, dt, 1e-5)
    W = _by_identity(H, G, D, V)
    for r in range(3):
        want = plain.attention(rows_in[r].astype(np.float32).astype(np.float64), W, "", m, 1e-5)
        np.testing.assert_allclose(got[r], want, atol=3e-5 if dtype == "float32" else 5e-2, rtol=1e-4 if dtype == "float32" else 3e-2)


@pytest.mark.parametrize("how, dtype, H, G, D, V", ATTENTION_CASES)
def test_one_key_far_away_stands_out(how, dtype, H, G, D, V):
    """Every query points at one key, whose value is marked: 0 to 300 tokens back, at page and tile borders, at the first
    tokens, in a portion and for a single token. The scale is small enough that only the temperature makes the key win, so a
    query with another position's temperature shows."""
    dt = getattr(torch, dtype)
    rng = np.random.default_rng(7)
    T = 321
    W = _by_identity(H, G, D, V)
    for mark in (0, 1, 15, 16, 63, 64, 127, 128, 300, 319):
        m = fu.left(H, G, D, V, (4.0, 40), scale=1.2 / D)
        x = np.zeros((T, (H + G) * D + G * V + H * V))
        x[:, :H * D] = np.tile(np.eye(D)[0] * 3.0, H)                              # after the norm: sqrt(D) along channel 0
        x[:, H * D:(H + G) * D] = np.tile(np.eye(D)[(1 if D > 1 else 0)], G)
        x[mark, H * D:(H + G) * D] = np.tile(np.eye(D)[0], G)
        x[mark, (H + G) * D:(H + G) * D + G * V] = 10.0 + np.arange(G * V)
        x[:, (H + G) * D + G * V:] = rng.standard_normal(H * V)                     # gates differ by channel and token
        for cuts in ([T], [T - 3, 1, 1, 1]) if how in ("rows", "tiles", "flash") else ([T - 20] + [1] * 20,):
            cache = _Pages([T], G, D, V, 16, dt, seed=mark)
            got = _run_attention(how, [[(0, k)] for k in cuts], [x], m, cache, dt, 1e-6)[0]
            want = plain.attention(x.astype(np.float32).astype(np.float64), W, "", m, 1e-6)
            tol = 1e-3 if dtype == "float32" else 0.03 * np.abs(want).max()
            np.testing.assert_allclose(got, want, atol=tol)


def test_the_temperature_changes_at_its_steps():
    """The queries as they are stored, at the positions around every step, for steps of 1, 7 and 64 positions."""
    from glassbox_b200 import kernels
    H, G, D, V = 2, 1, 6, 4
    rng = np.random.default_rng(5)
    for every in (1, 7, 64, 1000):
        positions = [0, 1, 5, 6, 7, 12, 13, 62, 63, 64, 126, 127, 128, 998, 999, 1000, 4095]
        n = len(positions)
        x = rng.standard_normal((n, (H + G) * D + G * V))
        q, k, v = torch.zeros((n, H * D), device=DEV), torch.zeros((2, G, 16, D), device=DEV), torch.zeros((2, G, 16, V), device=DEV)
        kernels.qk_norm_rope_write(_f32(x), None, None, None, _i32(positions), _i32(list(range(n))), q, k, v, H, G, D, V, 0, 1e-6, 16, True,
                                   _status(), unit_norm=True, q_temp=(0.3, every))
        unit = plain.rms_unit(x[:, :H * D].reshape(n, H, D), 1e-6)
        want = unit * np.array([plain.query_temperature(p, {"coef": 0.3, "every": every}) for p in positions])[:, None, None]
        np.testing.assert_allclose(q.view(n, H, D).cpu().numpy(), want, rtol=3e-6, atol=1e-6)
        keys = plain.rms_unit(x[:, H * D:(H + G) * D], 1e-6)
        np.testing.assert_allclose(k.permute(0, 2, 1, 3).reshape(-1, D)[:n].cpu().numpy(), keys, rtol=3e-6, atol=1e-6)


@pytest.mark.parametrize("n", [3, 300])
@pytest.mark.parametrize("E, top, groups, keep", [(8, 2, 4, 2), (6, 3, 3, 2), (5, 3, 1, 1), (1, 1, 1, 1), (16, 4, 2, 1), (64, 6, 8, 3), (4, 4, 2, 2)])
def test_router(n, E, top, groups, keep):
    from glassbox_b200 import kernels
    rng = np.random.default_rng(E + n)
    d = 40
    h, w = rng.standard_normal((n, d)), rng.standard_normal((E, d)) * 0.5
    choice, weight = torch.full((n, top), -7, dtype=torch.int32, device=DEV), torch.zeros((n, top), device=DEV)
    kernels.moe_route(_f32(h), _f32(w), None, None, _i32([0] * n), top, groups, keep, 1.0, choice, weight, None, softmax=True, group_best=True,
                      renorm_eps=1e-20)
    order, want = plain.route(h, {"router": w}, "", {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}})
    np.testing.assert_array_equal(choice.cpu().numpy(), order)
    np.testing.assert_allclose(weight.cpu().numpy(), want, atol=2e-6, rtol=2e-5)


def test_router_on_scores_made_by_hand():
    """A run wins by its best score alone (the sum of its two best would choose otherwise); experts of runs that are left out
    lose to smaller scores; logits so large that an unshifted exponential would overflow."""
    from glassbox_b200 import kernels
    s = np.array([0.30, 0.01, 0.20, 0.19, 0.02, 0.28])                             # best: 0.30, 0.20, 0.28; sums: 0.31, 0.39, 0.30
    for shift in (0.0, 200.0, -200.0):
        logits = np.log(s) + shift
        choice, weight = torch.zeros((1, 3), dtype=torch.int32, device=DEV), torch.zeros((1, 3), device=DEV)
        kernels.moe_route(_f32([[1.0, 0.0]]), _f32(np.stack([logits, np.zeros(6)], 1)), None, None, _i32([0]), 3, 3, 2, 1.0, choice, weight, None,
                          softmax=True, group_best=True, renorm_eps=1e-20)
        assert choice.tolist() == [[0, 5, 4]]
        np.testing.assert_allclose(weight.cpu().numpy()[0], np.array([0.30, 0.28, 0.02]) / 0.60, rtol=2e-4)


@pytest.mark.parametrize("n, dtype, form", [(5, "float32", "halves"), (5, "bfloat16", "halves"), (40, "bfloat16", "grouped"), (300, "bfloat16", "grouped")])
def test_swiglu_experts(n, dtype, form):
    from glassbox_b200 import kernels
    rng = np.random.default_rng(n)
    E, top, d, ff = 5, 2, 64, 40
    dt = getattr(torch, dtype)
    h = _rounded(rng.standard_normal((n, d)), dt)
    W = {}
    for e in range(E):
        for name, shape in (("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff))):
            W[f"e{e}.{name}"] = _rounded(rng.standard_normal(shape) / np.sqrt(shape[1]), dt)
    # gate row f and up row f are neighbours
    w_up = np.concatenate([np.stack([W[f"e{e}.gate"], W[f"e{e}.up"]], 1).reshape(2 * ff, d) for e in range(E)])
    w_down = np.concatenate([W[f"e{e}.down"] for e in range(E)])
    choice = np.stack([rng.permutation(E)[:top] for _ in range(n)])
    pair = torch.zeros((n, top * d), device=DEV)
    args = (_f32(h).to(dt), _f32(w_up).to(dt), _f32(w_down).to(dt), E, _i32(choice), _i32([0] * n))
    if form == "grouped":
        tables = torch.zeros(2 * (E + 1) + n * top, dtype=torch.int32, device=DEV)
        kernels.moe_experts_grouped(*args, tables, torch.zeros((n, top * ff), dtype=dt, device=DEV), pair, unit=kernels.SILU_UNIT)
    else:
        kernels.moe_expert_halves(*args, torch.zeros((n, top * ff), device=DEV), pair, unit=kernels.SILU_UNIT)
    got = pair.view(n, top, d).cpu().numpy()
    tol = 2e-5 if dtype == "float32" else 2e-2
    for r in range(n):
        for k in range(top):
            np.testing.assert_allclose(got[r, k], plain.expert(h[r], W, "", choice[r, k]), atol=tol, rtol=tol)


# ------------------------------------------------------------------------------------------------------ whole models
_MODELS = {}


def _model(name, tmp_path_factory, seed=21):
    key = (name, seed)
    if key not in _MODELS:
        cfg = fu.CONFIGS[name]()
        tensors = fu.random_weights(cfg, seed)
        folder = fu.write_model(str(tmp_path_factory.mktemp(f"fe_{name}_{seed}")), cfg, tensors)
        _MODELS[key] = (cfg, fu.as_float64(tensors), folder, {})
    return _MODELS[key]


def _want(model, tokens):
    cfg, W, _, memo = model
    key = tuple(tokens)
    if key not in memo:
        memo[key] = plain.forward(cfg, W, list(tokens))
    return memo[key]


def _tokens(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def _engine(folder, dtype, **kw):
    from glassbox_b200.engine.engine import Engine
    args = dict(cache_tokens=512, page_size=16, max_batch_tokens=256, max_requests=4)
    args.update(kw)
    return Engine(folder, dtype, **args)


@pytest.mark.parametrize("name", ["odd", "even", "ragged"])
def test_every_layer_of_a_short_request(name, tmp_path_factory):
    """The residual after every layer, in float32, against the plain one: the first layer that differs names itself."""
    cfg, W, folder, _ = _model(name, tmp_path_factory)
    eng = _engine(folder, "float32", use_graphs=False)
    toks = _tokens(cfg, 29, 4)
    layers, seen = [], []
    plain.forward(cfg, W, toks, layers)
    from glassbox_b200.engine.engine import StepEntry
    eng.add_request("r", [])

    def tapped(layer):
        inner = layer.forward

        def forward(ctx, x, *args, **kw):
            inner(ctx, x, *args, **kw)
            seen.append(x[:len(toks)].cpu().numpy().copy())
        return forward
    for layer in eng.model.layers:
        layer.forward = tapped(layer)
    try:
        eng.step([StepEntry("r", toks, [len(toks) - 1])])
    finally:
        for layer in eng.model.layers:
            del layer.forward
    assert len(seen) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(seen, layers)):
        np.testing.assert_allclose(a, b, atol=1e-4, rtol=1e-4, err_msg=f"after layer {i}")


@pytest.mark.parametrize("name, dtype", [(n, "float32") for n in sorted(fu.CONFIGS)] + [("odd", "bfloat16"), ("even", "bfloat16"), ("ragged", "bfloat16")])
def test_whole_prompt_and_token_by_token(name, dtype, tmp_path_factory):
    model = _model(name, tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, dtype)
    for n, seed in [(1, 1), (2, 2), (3, 6), (77, 3)]:                # the first tokens of a sequence; past several pages and a chunk
        toks = _tokens(cfg, n, seed)
        want = _want(model, toks)
        got = zu.run_schedule(eng, {"r": toks}, [[("r", n)]])["r"]
        assert_logits_close(got, want, dtype, f"{name} whole {n}")
        got = zu.run_schedule(eng, {"r": toks}, [[("r", 1)] for _ in range(n)])["r"]
        assert_logits_close(got, want, dtype, f"{name} token by token {n}")


@pytest.mark.parametrize("name, dtype", [("odd", "float32"), ("even", "float32"), ("ones", "float32"), ("even", "bfloat16")])
def test_portions_of_every_size(name, dtype, tmp_path_factory):
    model = _model(name, tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, dtype)
    toks = _tokens(cfg, 203, 7)
    want = _want(model, toks)
    for sizes in ([2] * 101 + [1], [3, 2, 16, 1, 15, 17, 2, 2, 63, 65, 17], [16] * 12 + [11], [31, 2, 33, 64, 64, 9], [1, 202]):
        assert sum(sizes) == len(toks)
        got = zu.run_schedule(eng, {"r": toks}, [[("r", k)] for k in sizes])["r"]
        assert_logits_close(got, want, dtype, f"{name} portions {sizes[:4]}...")


@pytest.mark.parametrize("name, dtype", [("odd", "float32"), ("even", "float32"), ("ragged", "float32"), ("even", "bfloat16")])
def test_mixed_batches_equal_each_request_alone(name, dtype, tmp_path_factory):
    """Unequal requests side by side, portions beside single tokens, requests that sit out a step, more requests than
    slots over time and a pool that only holds what is live: slots and pages are freed and used again."""
    model = _model(name, tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, dtype, cache_tokens=192, max_requests=3)
    reqs = {"a": _tokens(cfg, 70, 11), "b": _tokens(cfg, 9, 12), "c": _tokens(cfg, 33, 13), "d": _tokens(cfg, 50, 14),
            "e": _tokens(cfg, 1, 15), "f": _tokens(cfg, 18, 16)}
    schedule = [[("a", 30), ("b", 2)], [("b", 1), ("a", 2), ("c", 16)], [("a", 1), ("b", 1), ("c", 1)],
                [("c", 16), ("b", 5)],                              # b and c end: their slots and pages go back
                [("a", 1)], [("d", 20), ("a", 2)], [("e", 1), ("d", 1), ("a", 1)], [("d", 29), ("a", 1)],
                [("f", 2), ("a", 1)], [("f", 16), ("a", 25)]] + [[("a", 1)]] * 6
    want = {k: _want(model, v) for k, v in reqs.items()}
    got = zu.run_schedule(eng, reqs, schedule)
    for k in reqs:
        assert_logits_close(got[k], want[k], dtype, f"{name} mixed, request {k}")
    eng.cache.check_invariants()
    assert len(eng.cache.free_slots) == eng.cache.max_requests


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_single_tokens_in_front_of_a_portion(dtype, tmp_path_factory):
    """A mixed step whose head is single tokens takes the decoding kernel for them and the other form for the portion behind
    them, step after step, so that the recorded step is replayed as well."""
    model = _model("even", tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, dtype, cache_tokens=1024, max_requests=6)
    reqs = {c: _tokens(cfg, 20 + 8, 70 + i) for i, c in enumerate("abcde")}
    reqs["p"] = _tokens(cfg, 6 * 33 + 2, 80)
    schedule = [[(c, 20) for c in "abcde"]] + [[(c, 1) for c in "abcde"] + [("p", 33)] for _ in range(6)] + [[(c, 1) for c in "abcde"] + [("p", 1)]] * 2
    got = zu.run_schedule(eng, reqs, schedule)
    for k in reqs:
        assert_logits_close(got[k], _want(model, reqs[k]), dtype, f"request {k}")


def test_long_decoding_replays_recorded_steps(tmp_path_factory):
    """Two requests decode for more than two hundred steps: the steps run as recorded graphs, the states, the rings of the
    convolution's inputs and the pages carry from one replay to the next, the temperature passes its steps."""
    model = _model("even", tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, "float32", cache_tokens=512, max_requests=2)
    a, b = _tokens(cfg, 250, 31), _tokens(cfg, 226, 32)
    schedule = [[("a", 20)], [("b", 3)]] + [[("a", 1), ("b", 1)]] * 216 + [[("a", 14), ("b", 7)]]
    got = zu.run_schedule(eng, {"a": a, "b": b}, schedule)
    assert eng.graph_replays > 150
    assert_logits_close(got["a"], _want(model, a), "float32", "long decoding a")
    assert_logits_close(got["b"], _want(model, b), "float32", "long decoding b")
    eng.cache.check_invariants()


def test_a_slot_and_its_pages_that_are_used_again(tmp_path_factory):
    model = _model("odd", tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, "float32", max_requests=1, cache_tokens=64)
    for seed in (41, 42, 43):
        toks = _tokens(cfg, 40, seed)
        got = zu.run_schedule(eng, {"r": toks}, [[("r", 25)], [("r", 15)]])["r"]
        assert_logits_close(got, _want(model, toks), "float32", f"slot reuse {seed}")


def test_a_fork_carries_state_ring_and_pages(tmp_path_factory):
    from glassbox_b200.engine.engine import StepEntry
    model = _model("odd", tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, "float32")
    common, a, b = _tokens(cfg, 37, 91), _tokens(cfg, 6, 92), _tokens(cfg, 6, 93)
    eng.add_request("a", [])
    eng.step([StepEntry("a", common, [])])
    eng.fork("a", "b")
    got = {"a": [], "b": []}
    for x, y in zip(a, b):
        rows = eng.step([StepEntry("a", [x], [0]), StepEntry("b", [y], [0])]).float().cpu().numpy()
        got["a"].append(rows[0])
        got["b"].append(rows[1])
    for k, tail in (("a", a), ("b", b)):
        assert_logits_close(np.array(got[k]), _want(model, common + tail)[37:], "float32", f"fork {k}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(dtype, tmp_path_factory):
    import glassbox_b200
    model = _model("even", tmp_path_factory, seed=5)
    cfg, W, folder, _ = model
    llm = glassbox_b200.load(folder, dtype, blocks=64, budget=32, max_seqs=3, prefix_cache=True)
    prompts = [_tokens(cfg, 37, 51), _tokens(cfg, 5, 52), _tokens(cfg, 70, 53), _tokens(cfg, 1, 54)]
    outs = llm.generate(prompts, max_tokens=10)
    for p, out in zip(prompts, outs):
        seq = list(p)
        assert len(out) == 10
        for i, tok in enumerate(out):
            logits = plain.forward(cfg, W, seq)[-1]
            best = int(np.argmax(logits))
            if dtype == "bfloat16" and tok != best:
                top2 = np.sort(logits)[-2:]
                assert logits[tok] >= top2[1] - 0.3 * logits.std(), f"token {i}: {tok} is not near the best"
                break                                                # rounding chose the runner-up: the texts part ways
            assert tok == best, f"{dtype} prompt of {len(p)}: token {i} is {tok}, plain says {best}"
            seq.append(tok)


def test_a_trace_replayed_from_the_command_line(tmp_path_factory, tmp_path):
    """``bin/trace_run`` as a user runs it: steps on standard input, logits in files; four live requests at most in a pool that
    holds only what is live, portions beside single tokens, requests that end and others that take their slots and pages."""
    import json
    import os
    import subprocess
    import sys
    from replay_util import TRACE_RUN, live_tokens_needed
    model = _model("odd", tmp_path_factory)
    cfg, _, folder, _ = model
    reqs = {"a": _tokens(cfg, 150, 61), "b": _tokens(cfg, 40, 62), "c": _tokens(cfg, 66, 63), "d": _tokens(cfg, 9, 64), "e": _tokens(cfg, 70, 65)}
    plan = [[("a", 64), ("b", 2)], [("a", 3), ("b", 1), ("c", 29)], [("a", 1), ("b", 16), ("c", 1), ("d", 2)],
            [("a", 16), ("b", 21), ("c", 36), ("d", 7)], [("a", 1), ("e", 64)], [("a", 64), ("e", 2)], [("a", 1), ("e", 4)]]
    at, steps = {k: 0 for k in reqs}, []
    for i, step in enumerate(plan):
        entries, end = [], []
        for rid, k in step:
            entries.append({"id": rid, "tokens": reqs[rid][at[rid]:at[rid] + k], "want": list(range(k))})
            at[rid] += k
            if at[rid] == len(reqs[rid]):
                end.append(rid)
        steps.append({"step": i, "entries": entries, "end": end})
    assert at == {k: len(v) for k, v in reqs.items()}
    out = str(tmp_path / "out")
    os.makedirs(out)
    proc = subprocess.run([sys.executable, TRACE_RUN, "--model", folder, "--dtype", "float32", "--out", out, "--max-tokens",
                           str(live_tokens_needed(steps))], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                          text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(plan))]
    got = {k: [] for k in reqs}
    for i, step in enumerate(plan):
        rows = np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])
        row = 0
        for rid, k in step:
            got[rid].append(rows[row:row + k])
            row += k
        assert row == len(rows)
    for rid in reqs:
        assert_logits_close(np.concatenate(got[rid], 0), _want(model, reqs[rid]), "float32", f"replayed request {rid}")
