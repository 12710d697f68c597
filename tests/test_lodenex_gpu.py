"""Lodenex on the GPU against the plain float64 implementation (``tests/plain/lodenex_plain.py``): each mechanism's kernels
alone, then whole models under every way of cutting and batching their requests, through the engine's own step function,
cache manager, scheduler and entry point. Sizes are the tests' own (``lodenex_util.CONFIGS``)."""
import math

import numpy as np
import pytest
import torch

import conftest
from plain import lodenex_plain as plain
import lodenex_util as lu
import zurerax_util as zu
from test_felovik_gpu import _cuts, _f32, _gather, _i32, _Pages, _rounded, _scatter, _status, _step_meta

pytestmark = pytest.mark.gpu
DEV = "cuda:0"

# bfloat16 against float64 on sharp models (the largest seen: 0.10 and 0.006 of the spread). Faults in which
# key or token a bfloat16 kernel reads are caught by the crafted tests below and by the float32 runs of the same code, which are
# held to 1e-4.
BF16_REL_MAX, BF16_REL_MEAN = 0.2, 0.012


def assert_logits_close(got, want, dtype, what=""):
    if dtype == "float32":
        return conftest.assert_logits_close(got, want, dtype, what)
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all(), what
    diff, spread = np.abs(got - want), want.std()
    assert diff.max() <= BF16_REL_MAX * spread, f"{what}: max abs diff {diff.max():.3e} > {BF16_REL_MAX} x spread {spread:.3e}"
    assert diff.mean() <= BF16_REL_MEAN * spread, f"{what}: mean abs diff {diff.mean():.3e} > {BF16_REL_MEAN} x spread {spread:.3e}"


def _freqs(values):
    return _f32(values)


# ------------------------------------------------------------------------------- between the projection and the attention
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n, H, G, D, V, rot", [(5, 4, 2, 16, 8, 16), (1, 1, 1, 2, 1, 2), (7, 3, 1, 9, 7, 6), (300, 6, 3, 20, 12, 8), (4, 8, 2, 64, 64, 64),
                                                (3, 5, 5, 96, 96, 32), (400, 2, 1, 6, 4, 2), (2, 32, 8, 128, 128, 96), (6, 2, 2, 10, 10, 0)])
def test_norm_over_the_projection_rotation_and_cache_write(dtype, n, H, G, D, V, rot):
    """Queries and keys normed over all heads at once, rotated in halves at positions up to far ones, stored at scattered slots;
    padding rows are left alone, other slots too, and nothing is stored when the run does not write."""
    from glassbox_b200 import kernels
    rng = np.random.default_rng(n + D)
    dt, page, pages = getattr(torch, dtype), 16, -(-n // 16) + 2
    cols = (H + G) * D + G * V
    x = rng.standard_normal((n, cols)).astype(np.float32).astype(np.float64)
    gq, gk = 1 + 0.3 * rng.standard_normal(H * D), 1 + 0.3 * rng.standard_normal(G * D)
    positions = [int(p) for p in rng.integers(0, 5000, n)]
    if n > 2:
        positions[1] = -1
    slots = [int(s) for s in rng.permutation(pages * page)[:n]]
    freqs, length = plain.frequencies_by_wavelength(rot, 500.0, lu.bands(3.0, 100, 1.0, 4.0)) if rot else ([], 1.0)
    freqs = [float(np.float32(f)) for f in freqs]
    proj = torch.full((n, cols + 5), 50.0, device=DEV)
    for off in (0, 4, 5):                                           # rows that start 8-byte aligned, and rows that do not
        buf = torch.full((n, cols + 5), 50.0, device=DEV)
        proj = buf[:, off:off + cols]
        proj.copy_(_f32(x))
        q = torch.full((n, H * D), 7.0, dtype=dt, device=DEV)
        k, v = torch.full((pages, G, page, D), 7.0, dtype=dt, device=DEV), torch.full((pages, G, page, V), 7.0, dtype=dt, device=DEV)
        status = _status()
        args = (_f32(gq), _f32(gk), _freqs(freqs) if rot else None, 1.25, _i32(positions), _i32(slots), q, k, v, H, G, D, V, rot, 1e-5, page)
        kernels.projection_norm_rope_write(proj, *args, False, status)
        assert bool((k == 7.0).all()) and bool((v == 7.0).all())
        q.fill_(7.0)
        kernels.projection_norm_rope_write(proj, *args, True, status)
        assert int(status.item()) == 0
        wq = plain.rms(x[:, :H * D], gq, 1e-5).reshape(n, H, D)
        wk = plain.rms(x[:, H * D:(H + G) * D], gk, 1e-5).reshape(n, G, D)
        wv = x[:, (H + G) * D:].reshape(n, G, V)
        kn, vn = k.float().cpu().numpy(), v.float().cpu().numpy()
        tol = dict(atol=6e-4, rtol=1e-4) if dtype == "float32" else dict(atol=3e-2, rtol=1e-2)      # (angles of thousands of radians in float32)
        for r in range(n):
            if positions[r] < 0:
                assert bool((q[r] == 7.0).all()) and (kn[slots[r] // page, :, slots[r] % page] == 7.0).all()
                continue
            turn = lambda t: plain.rotate(t, positions[r], freqs, 1.25)
            np.testing.assert_allclose(q[r].float().cpu().numpy().reshape(H, D), turn(wq[r]), **tol)
            np.testing.assert_allclose(kn[slots[r] // page, :, slots[r] % page], turn(wk[r]), **tol)
            np.testing.assert_allclose(vn[slots[r] // page, :, slots[r] % page], wv[r], **tol)
        used = np.zeros((pages, page), dtype=bool)
        for r in range(n):
            used[slots[r] // page, slots[r] % page] |= positions[r] >= 0
        assert (kn.transpose(0, 2, 1, 3)[~used] == 7.0).all() and (vn.transpose(0, 2, 1, 3)[~used] == 7.0).all()
        if rot == 0:
            kernels.projection_norm_rope_write(proj, None, None, *args[2:], True, status)              # no norm at all
            live = torch.tensor([p >= 0 for p in positions])
            np.testing.assert_allclose(q[live].float().cpu().numpy(), x[live.numpy(), :H * D], atol=2e-2)


def test_a_slot_outside_the_cache_is_reported_and_skipped():
    from glassbox_b200 import kernels
    x, status = torch.ones((2, 8), device=DEV), _status()
    q, k, v = torch.zeros((2, 4), device=DEV), torch.full((1, 1, 4, 2), 7.0, device=DEV), torch.full((1, 1, 4, 2), 7.0, device=DEV)
    kernels.projection_norm_rope_write(x, None, None, None, 1.0, _i32([0, 1]), _i32([4, -1]), q, k, v, 2, 1, 2, 2, 0, 1e-5, 4, True, status)
    assert int(status.item()) == 2 and bool((k == 7.0).all()) and bool((v == 7.0).all())
    status = _status()
    lat, cq, cache = torch.ones((1, 9), device=DEV), torch.zeros((1, 3), device=DEV), torch.full((1, 1, 4, 6), 7.0, device=DEV)
    kernels.latent_inputs(lat, torch.ones(3, device=DEV), torch.ones(4, device=DEV), torch.zeros(1, device=DEV), 1.0, _i32([0]), _i32([9]), cq, cache,
                          4, 2, 2, 1e-5, True, status)
    assert int(status.item()) == 2 and bool((cache == 7.0).all()) and cq[0].tolist() == pytest.approx([1.0] * 3, rel=1e-4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n, qr, c, r, rot", [(5, 24, 16, 8, 8), (1, 1, 1, 2, 2), (9, 13, 22, 6, 4), (40, 512, 128, 64, 64), (3, 1536, 512, 64, 64)])
def test_latent_inputs(dtype, n, qr, c, r, rot):
    from glassbox_b200 import kernels
    rng = np.random.default_rng(qr + c)
    dt, page = getattr(torch, dtype), 16
    x = rng.standard_normal((n, qr + c + r)).astype(np.float32).astype(np.float64)
    gq, gl = 1 + 0.3 * rng.standard_normal(qr), 1 + 0.3 * rng.standard_normal(c)
    positions, slots = [int(p) for p in rng.integers(0, 900, n)], [int(s) for s in rng.permutation(64)[:n]]
    if n > 2:
        positions[2] = -1
    freqs, length = plain.frequencies_by_turns(rot, 300.0, lu.ramp(3.0, 200, 8.0, 1.0))
    cq, cache, status = torch.full((n, qr), 7.0, dtype=dt, device=DEV), torch.full((4, 1, page, c + r), 7.0, dtype=dt, device=DEV), _status()
    buf = torch.full((n, qr + c + r + 3), 50.0, device=DEV)
    buf[:, :qr + c + r] = _f32(x)
    args = (_f32(gq), _f32(gl), _freqs(freqs), length, _i32(positions), _i32(slots), cq, cache, c, r, rot, 1e-6)
    kernels.latent_inputs(buf[:, :qr + c + r], *args, False, status)
    assert bool((cache == 7.0).all())
    kernels.latent_inputs(buf[:, :qr + c + r], *args, True, status)
    assert int(status.item()) == 0
    got, rows = cq.float().cpu().numpy(), cache.float().cpu().numpy().reshape(64, c + r)
    tol = dict(atol=2e-4, rtol=1e-4) if dtype == "float32" else dict(atol=3e-2, rtol=1e-2)
    for i in range(n):
        if positions[i] < 0:
            assert not got[i].any() and (rows[slots[i]] == 7.0).all()
            continue
        np.testing.assert_allclose(got[i], plain.rms(x[i, :qr], gq, 1e-6), **tol)
        np.testing.assert_allclose(rows[slots[i], :c], plain.rms(x[i, qr:qr + c], gl, 1e-6), **tol)
        np.testing.assert_allclose(rows[slots[i], c:], plain.rotate(x[i, qr + c:], positions[i], freqs, length), **tol)
    left = [s for s in range(64) if s not in slots]
    assert (rows[left] == 7.0).all()


@pytest.mark.parametrize("H, dq, r, rot, c", [(3, 10, 6, 6, 22), (2, 16, 9, 4, 8), (4, 32, 16, 16, 64), (5, 64, 32, 8, 128)])
def test_the_query_rotation_in_halves(H, dq, r, rot, c):
    """Alone, in both dtypes, and carried by the per-head product that forms the rest of the query."""
    from glassbox_b200 import kernels
    rng = np.random.default_rng(H + dq)
    n = 70
    freqs, length = plain.frequencies_by_turns(rot, 300.0, lu.ramp(3.0, 200, 8.0, 1.0))
    positions = [int(p) for p in rng.integers(0, 900, n)]
    positions[3] = -1
    for dtype in (torch.float32, torch.bfloat16):
        x = _rounded(rng.standard_normal((n, H * (dq + r))), dtype)
        w = _rounded(rng.standard_normal((H, c, dq)) / np.sqrt(dq), dtype)
        q, qabs, cache = _f32(x).to(dtype), torch.full((n, H * (c + r)), 7.0, dtype=dtype, device=DEV), torch.zeros((1, 1, 16, c + r), dtype=dtype, device=DEV)
        kernels.latent_kv_write(q, 0, qabs, cache, None, _freqs(freqs), _i32(positions), _i32([0] * n), H, dq, r, c, rot, 1e-6, False, _status(),
                                half_pairs=True, magnitude=length)
        forms = [qabs.float().cpu().numpy().reshape(n, H, c + r)]
        if dtype == torch.bfloat16 and kernels.head_linear_supported(q, _f32(w).to(dtype), qabs, dq + r, c + r):
            fused = torch.full_like(qabs, 7.0)
            kernels.head_linear(q, _f32(w).to(dtype), fused, dq + r, c + r, turn=(_i32(positions), _freqs(freqs), length, rot, r))
            f = fused.float().cpu().numpy().reshape(n, H, c + r)
            np.testing.assert_allclose(f[:, :, :c], np.einsum("nhk,hck->nhc", x.reshape(n, H, dq + r)[:, :, :dq], w), atol=3e-2, rtol=2e-2)
            forms.append(f)
        for f in forms:
            assert (f[3, :, c:] == 7.0).all() and (len(forms) == 2 or (f[:, :, :c] == 7.0).all() or f is not forms[0])
            for i in range(n):
                if positions[i] >= 0:
                    np.testing.assert_allclose(f[i, :, c:], plain.rotate(x[i].reshape(H, dq + r)[:, dq:], positions[i], freqs, length),
                                               atol=2e-4 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("n, heads, N, K", [(1, 3, 40, 16), (70, 6, 128, 64), (200, 16, 64, 128), (33, 2, 130, 256), (65, 2, 6, 32)])
@pytest.mark.parametrize("gate_dtype, off", [(torch.float32, 0), (torch.float32, 1), (torch.bfloat16, 3)])
def test_a_gate_per_channel_behind_the_per_head_product(n, heads, N, K, gate_dtype, off):
    from glassbox_b200 import kernels
    g = torch.Generator(device="cpu").manual_seed(n + N)
    a = torch.randn((n, heads * K), generator=g).to(torch.bfloat16).to(DEV)
    w = (torch.randn((heads, N, K), generator=g) / K ** 0.5).to(torch.bfloat16).to(DEV)
    gate = (torch.randn((n, heads * N + 4), generator=g) * 2).to(gate_dtype).to(DEV)[:, off:off + heads * N]
    out = torch.full((n, heads * N), 9.0, dtype=torch.bfloat16, device=DEV)
    kernels.head_linear(a, w, out, K, N, gate=gate)
    want = torch.einsum("nhk,hck->nhc", a.float().view(n, heads, K), w.float()).reshape(n, -1) * torch.sigmoid(gate.float())
    assert torch.allclose(out.float(), want, atol=0.03, rtol=0.02)
    # the same gate as a kernel of its own, where the product has no epilogue for it
    for dtype in (torch.float32, torch.bfloat16):
        y = torch.randn((n, heads * N), generator=g).to(dtype).to(DEV)
        want = y.double() * torch.sigmoid(gate.double())
        kernels.gate_rows_(y, gate)
        assert torch.allclose(y.double(), want, atol=1e-6 if dtype == torch.float32 else 2e-2, rtol=1e-5 if dtype == torch.float32 else 1e-2)


# -------------------------------------------------------------------------------------------------- pointwise functions
def test_gelu_alone_and_in_the_products_epilogues():
    from glassbox_b200 import kernels
    z = np.concatenate([np.linspace(-12, 12, 4001), [0.0, 1e-6, -1e-6, 40.0, -40.0, 1e4, -1e4]])
    for dtype in (torch.float32, torch.bfloat16):
        out = torch.zeros((1, len(z)), dtype=dtype, device=DEV)
        kernels.gelu(_f32(z[None]), out)
        np.testing.assert_allclose(out.float().cpu().numpy()[0], plain.gelu(z), atol=1e-6, rtol=2e-6 if dtype == torch.float32 else 5e-3)
    g = torch.Generator(device="cpu").manual_seed(3)
    for rows, ff, d in ((5, 272, 128), (64, 48, 64), (200, 272, 128), (130, 64, 72)):
        a = (2 * torch.randn((rows, d), generator=g)).to(torch.bfloat16).to(DEV)
        w = (torch.randn((ff, d), generator=g) / d ** 0.5).to(torch.bfloat16).to(DEV)
        want = plain.gelu((a.double() @ w.double().T).cpu().numpy())
        got = torch.zeros((rows, ff), dtype=torch.bfloat16, device=DEV)
        (kernels.gemm_stream if rows <= kernels.STREAM_MAX_ROWS else kernels.gemm_tc)(a, w, got, gelu=True)
        np.testing.assert_allclose(got.float().cpu().numpy(), want, atol=2e-3, rtol=8e-3)


@pytest.mark.parametrize("shape", [(1, 1), (3, 7), (5, 1000), (2, 4099)])
def test_capped_logits(shape):
    from glassbox_b200 import kernels
    x = np.random.default_rng(0).standard_normal(shape) * 30
    x.flat[0] = 1e6
    for cap in (1.0, 15.0, 50.0):
        t = _f32(x)
        kernels.tanh_cap_(t, cap)
        np.testing.assert_allclose(t.cpu().numpy(), plain.tanh_cap(x, cap), atol=2e-6 * cap, rtol=2e-6)


# ---------------------------------------------------------------------------------- capped attention within chunks
def _run_attention(how, steps, qkv, gates, cache, dtype, H, G, D, V, scale, cap, sink, chunk, window=None):
    """Queries into a buffer and keys and values into the cache as they are, then attention with its gate, step by step. ``how``:
    "rows", "decode" and "split" (the two kernels for single tokens; portions take the row kernel), "tiles" or "flash"."""
    from glassbox_b200 import kernels
    page, cols = cache.page, (H + G) * D + G * V
    got = [np.zeros((len(r), H * V)) for r in qkv]
    at = [0] * len(qkv)
    status = _status()
    sk = _f32(sink) if sink is not None else None
    own = dict(softcap=cap, chunk=chunk)
    common = dict(r1=None, r2=None, sink=sk, heads=H, kv_heads=G, dim=D, vdim=V, page_size=page, scale=scale, window=window, status=status, **own)
    for step in steps:
        n, row_seq, positions, first, start = _step_meta(step, at)
        proj = _f32(_gather(step, at, qkv, cols))
        slots = [s for e in step for s in ([-1] if e is None else [cache.slot(e[0], at[e[0]] + i) for i in range(e[1])])]
        gate = _f32(_gather(step, at, gates, H)) if gates is not None else None
        q, out = torch.zeros((n, H * D), dtype=dtype, device=DEV), torch.zeros((n, H * V), dtype=dtype, device=DEV)
        kernels.projection_norm_rope_write(proj, None, None, None, 1.0, positions, _i32(slots), q, cache.k, cache.v, H, G, D, V, 0, 1e-6, page, True,
                                           status)
        tables = []
        for e in step:
            row = [-1] * cache.width if e is None else list(cache.row(e[0]))
            if e is not None:
                # pages that no row of this step sees are given back, as the cache manager does
                lo = at[e[0]] // chunk * chunk if chunk else max(0, at[e[0]] - window + 1) if window else 0
                row[:lo // page] = [-1] * (lo // page)
            tables.append(row)
        tables = _i32(tables)
        single = all(e is None or e[1] == 1 for e in step)
        longest = max(e[1] for e in step if e)
        if how == "flash":
            kernels.attention_prefill_tc(q, out, cache.k, cache.v, tables, first, start, longest, H, G, D, page, scale, window, status,
                                         sink_terms=(None, None, sk, gate), **own)
        elif how == "tiles":
            kernels.sink_attention_tiles(q, out, cache.k, cache.v, tables, first, start, longest, gate=gate, **common)
        elif how == "split" and single:
            plans = [(1, 0, 4), (3, 16, 4), (2, 16, 8), (2, 0, 8), (5, 0, 4)] if D == 64 else [(1, 0, 4), (3, 0, 4), (2, 0, 4)]
            splits, block_keys, warps = plans[sum(at) % len(plans)]
            part_acc = torch.full((n, H * warps * splits * D), float("nan"), device=DEV)
            part_ml = torch.full((n, H * warps * splits * 2), float("nan"), device=DEV)
            counters = torch.zeros(n * G, dtype=torch.int32, device=DEV)
            kernels.attention_decode_mma(q, out, cache.k, cache.v, tables, row_seq, positions, H, G, D, page, scale, window, splits, part_acc,
                                         part_ml, counters, status, block_keys, warps, sink_terms=(None, None, sk, gate), **own)
        elif how == "decode" and single:
            kernels.sink_attention_decode(q, out, cache.k, cache.v, tables, row_seq, positions, gate=gate, **common)
        else:
            kernels.sink_attention_rows(q, out, cache.k, cache.v, tables, row_seq, positions, gate=gate, **common)
        _scatter(step, at, out.float().cpu().numpy(), got)
    assert int(status.item()) == 0
    return got


def _plain_attention(qkv, gates, dtype, H, G, D, V, scale, cap, sink, chunk):
    x = _rounded(qkv, dtype)
    T = len(x)
    out = plain.capped_attention(x[:, :H * D].reshape(T, H, D), x[:, H * D:(H + G) * D].reshape(T, G, D), x[:, (H + G) * D:].reshape(T, G, V), scale,
                                 cap, sink, chunk)
    if gates is not None:
        out = out * plain.logistic(gates)[:, :, None]
    return out.reshape(T, H * V)


ATTENTION_CASES = [("rows", "float32", 6, 2, 20, 12), ("rows", "float32", 3, 1, 9, 7), ("decode", "float32", 4, 2, 16, 32), ("decode", "bfloat16", 8, 2, 48, 64),
                   ("split", "bfloat16", 8, 2, 64, 64), ("split", "bfloat16", 4, 4, 32, 32), ("split", "bfloat16", 4, 2, 128, 128),
                   ("split", "bfloat16", 6, 2, 96, 96), ("tiles", "bfloat16", 4, 2, 64, 32), ("tiles", "bfloat16", 2, 1, 128, 128),
                   ("tiles", "bfloat16", 2, 1, 80, 80), ("tiles", "bfloat16", 2, 2, 96, 96), ("flash", "bfloat16", 4, 2, 64, 64)]


@pytest.mark.parametrize("chunk, cap, with_sink, with_gate", [(40, 3.0, True, True), (None, 2.0, True, False), (64, None, False, True), (7, 5.0, True, True),
                                                              (1, 1.0, True, True)])
@pytest.mark.parametrize("how, dtype, H, G, D, V", ATTENTION_CASES)
def test_attention_in_portions_over_scattered_pages(how, dtype, H, G, D, V, chunk, cap, with_sink, with_gate):
    rng = np.random.default_rng(H * D + V)
    dt = getattr(torch, dtype)
    lengths = [150, 21, 67]
    cols = (H + G) * D + G * V
    qkv, gates = [rng.standard_normal((n, cols)) for n in lengths], [rng.standard_normal((n, H)) for n in lengths]
    gates = [g.astype(np.float32).astype(np.float64) for g in gates] if with_gate else None
    sink = rng.standard_normal(H) * 2 if with_sink else None
    scale = 2.0 / math.sqrt(D)
    got = _run_attention(how, _cuts(lengths, rng), qkv, gates, _Pages(lengths, G, D, V, 16, dt), dt, H, G, D, V, scale, cap, sink, chunk)
    for r in range(3):
        want = _plain_attention(qkv[r], gates[r] if gates else None, dt, H, G, D, V, scale, cap, sink, chunk)
        np.testing.assert_allclose(got[r], want, atol=3e-5 if dtype == "float32" else 4e-2, rtol=1e-4 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("how, dtype, H, G, D, V", ATTENTION_CASES)
def test_one_key_stands_out_just_inside_and_just_outside_a_chunk(how, dtype, H, G, D, V):
    """Every query points at one key, whose value is marked: the first and the last of a chunk, at page and tile borders, at the
    first tokens; rows of the same chunk see it (to within the sink and the cap), rows of the next do not."""
    dt, T, scale, cap = getattr(torch, dtype), 300, 1.0, 9.0
    cols = (H + G) * D + G * V
    for chunk in (48, 100, 128):
        for mark in (0, 1, 15, 16, 47, 48, 63, 64, 95, 99, 100, 127, 128, 199, 255, 256, 299):
            x = np.zeros((T, cols))
            x[:, :H * D] = np.tile(np.eye(D)[0] * 8.0, H)
            x[mark, H * D:(H + G) * D] = np.tile(np.eye(D)[0] * 8.0, G)              # score 64: capped to about 9
            x[mark, (H + G) * D:] = 10.0 + np.arange(G * V) % 7
            cuts = ([T], [T - 3, 1, 1, 1]) if how in ("rows", "tiles", "flash") else ([T - 20] + [1] * 20,)
            if how in ("decode", "split") and (mark // chunk + 1) * chunk < T - 20:
                cuts = ([mark + 1] + [1] * min(12, T - mark - 1) + [max(T - mark - 13, 0)],)     # decode right behind the marked key
                cuts = ([k for k in cuts[0] if k],)
            for cut in cuts:
                got = _run_attention(how, [[(0, k)] for k in cut], [x], None, _Pages([T], G, D, V, 16, dt, seed=mark), dt, H, G, D, V, scale, cap,
                                     np.zeros(H), chunk)[0]
                want = _plain_attention(x, None, dt, H, G, D, V, scale, cap, np.zeros(H), chunk)
                seen = [t for t in range(T) if t >= mark and t // chunk == mark // chunk]
                assert (want[seen] > 9.0).all() and not want[[t for t in range(T) if t not in seen]].any()
                np.testing.assert_allclose(got, want, atol=1e-3 if dtype == "float32" else 0.1)


@pytest.mark.parametrize("how, dtype, H, G, D, V", [c for c in ATTENTION_CASES if c[0] != "rows" or c[4] == 20])
def test_the_cap_and_the_sink_in_closed_form(how, dtype, H, G, D, V):
    """All scores equal and far above, near and far below the cap: each weighs 1 / (keys + exp(sink - capped score))."""
    dt, T, chunk = getattr(torch, dtype), 90, 32
    cols = (H + G) * D + G * V
    sink = np.linspace(-4.0, 6.0, H)
    for score, cap in ((1000.0, 4.0), (-1000.0, 3.0), (2.0, 4.0), (-0.5, 1.0), (1e-3, 8.0)):
        x = np.zeros((T, cols))
        x[:, :H * D] = np.tile(np.eye(D)[0], H)
        x[:, H * D:(H + G) * D] = np.tile(np.eye(D)[0], G)
        x[:, (H + G) * D:] = 1.0
        got = _run_attention(how, [[(0, 70)]] + [[(0, 1)]] * 20, [x], None, _Pages([T], G, D, V, 16, dt), dt, H, G, D, V, score, cap, sink, chunk)[0]
        s = cap * math.tanh(score / cap)
        for t in range(T):
            keys = t % chunk + 1
            want = np.repeat(keys / (keys + np.exp(sink - s)), V)
            np.testing.assert_allclose(got[t], want, atol=2e-5 if dtype == "float32" else 6e-3)


# ------------------------------------------------------------------------------------------- latent attention in a window
@pytest.mark.parametrize("how, dtype, H, c, r", [("rows", "float32", 3, 22, 6), ("rows", "bfloat16", 2, 13, 5), ("mma", "bfloat16", 3, 64, 16),
                                                 ("mma", "bfloat16", 16, 128, 32), ("mma", "bfloat16", 20, 128, 64)])
def test_one_latent_stands_out_just_inside_and_just_outside_the_window(how, dtype, H, c, r):
    """Portions cut at changing places and single tokens (the keys in several shares): a marked token is read by exactly the rows
    whose window holds it. Pages behind the window are gone."""
    from glassbox_b200 import kernels
    dt, T, page, w = getattr(torch, dtype), 260, 16, c + r
    width = -(-T // page)
    for window, mark in [(1, 70), (13, 0), (13, 64), (40, 63), (40, 127), (64, 16), (64, 191), (100, 31), (150, 100), (1000, 5)]:
        rng = np.random.default_rng(mark)
        order = rng.permutation(width + 3)[:width]
        cache = torch.zeros((width + 3, 1, page, w), dtype=dt, device=DEV)
        rows = np.zeros((T, w))
        rows[mark, :c] = 3.0 + np.arange(c) % 5
        rows[mark, c] = 1.0
        for t in range(T):
            cache[int(order[t // page]), 0, t % page] = _f32(rows[t]).to(dt)
        at, status = 0, _status()
        for k in [50, 2, 3, 64, 65] + [1] * 8 + [40] + [1] * 28:
            q = torch.zeros((k, H, w), dtype=dt, device=DEV)
            q[:, :, c] = 12.0                                        # the marked token scores 12, all others 0
            table = [int(p) for p in order]
            gone = max(0, at - window + 1) // page
            table[:gone] = [-1] * gone
            table = _i32([table])
            out = torch.full((k, H * c), 7.0, dtype=dt, device=DEV)
            q = q.reshape(k, -1)
            positions = _i32(list(range(at, at + k)))
            if how == "rows":
                kernels.latent_attention_rows(q, out, cache, table, _i32([0] * k), positions, None, H, c, r, page, 1.0, window, status)
            elif k == 1:
                shares = 1 + at % 4
                part_o, part_ml = torch.zeros((1, H * shares * c), device=DEV), torch.zeros((1, H * shares * 2), device=DEV)
                kernels.latent_attention_mma(q, out, cache, table, _i32([0, 1]), positions, positions, None, H, c, r, page, 1.0, window, status,
                                             decode=True, splits=shares, part_o=part_o, part_ml=part_ml)
            else:
                kernels.latent_attention_mma(q, out, cache, table, _i32([0, k]), _i32([at]), positions, None, H, c, r, page, 1.0, window, status,
                                             max_rows_per_seq=k)
            got = out.float().cpu().numpy().reshape(k, H, c)
            for i in range(k):
                keys = plain.window_keys(at + i, window)
                want = np.zeros(c)
                if mark in keys:
                    want = rows[mark, :c] * math.exp(12.0) / (math.exp(12.0) + len(keys) - 1)
                np.testing.assert_allclose(got[i], np.tile(want, (H, 1)), atol=1e-4 if dtype == "float32" else 4e-2, err_msg=f"window {window} mark {mark} row {at + i}")
            at += k
        assert int(status.item()) == 0


# ------------------------------------------------------------------------------------------------------ whole models
_MODELS = {}


def _model(name, tmp_path_factory, seed=21):
    key = (name, seed)
    if key not in _MODELS:
        cfg = lu.CONFIGS[name]()
        tensors = lu.random_weights(cfg, seed)
        folder = lu.write_model(str(tmp_path_factory.mktemp(f"lo_{name}_{seed}")), cfg, tensors)
        _MODELS[key] = (cfg, lu.as_float64(tensors), folder, {})
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
    toks = _tokens(cfg, 59, 4)
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


@pytest.mark.parametrize("name, dtype", [(n, "float32") for n in sorted(lu.CONFIGS)] + [("odd", "bfloat16"), ("even", "bfloat16"), ("ragged", "bfloat16")])
def test_whole_prompt_and_token_by_token(name, dtype, tmp_path_factory):
    model = _model(name, tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, dtype)
    for n, seed in [(1, 1), (2, 2), (3, 6), (77, 3)]:                # the first tokens of a sequence; past several pages and chunks
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
    for sizes in ([2] * 101 + [1], [3, 2, 16, 1, 15, 17, 2, 2, 63, 65, 17], [23] * 8 + [19], [31, 2, 33, 64, 64, 9], [1, 202], [48, 48, 48, 48, 11]):
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
    for g in range(len(eng.cache.groups)):
        assert eng.cache.free_pages(g) == eng.cache.num_pages(g)


def test_chunks_hold_no_more_pages_than_the_current_one_needs(tmp_path_factory):
    """A long request lives in groups whose pools are far smaller than it: pages come back at the chunk's end or behind the window
    and are used again by the same request, and by its neighbour."""
    cfg = lu.config(97, 32, [lu.layer(lu.attention(2, 1, 8, 8, 4, chunk=24), 16), lu.layer(lu.latent(2, 8, 4, 8, 8, 8, window=20), None),
                             lu.layer(lu.attention(2, 2, 8, 8, 8, chunk=32), None)])
    tensors = lu.random_weights(cfg, 3)
    folder = lu.write_model(str(tmp_path_factory.mktemp("lo_small")), cfg, tensors)
    model = (cfg, lu.as_float64(tensors), folder, {})
    eng = _engine(folder, "float32", max_requests=2, group_pages=lambda spec: 8, max_batch_tokens=64)
    reqs = {"a": _tokens(cfg, 300, 1), "b": _tokens(cfg, 170, 2)}
    schedule = [[("a", 40)], [("a", 1), ("b", 30)]] + [[("a", 1), ("b", 1)]] * 130 + [[("a", 20), ("b", 10)]] + [[("a", 9)]] * 12 + [[("a", 1)]]
    got = zu.run_schedule(eng, reqs, schedule)
    for k in reqs:
        assert_logits_close(got[k], _want(model, reqs[k]), "float32", f"request {k}")
    eng.cache.check_invariants()
    assert all(eng.cache.free_pages(g) == 8 for g in range(3))


def test_long_decoding_replays_recorded_steps(tmp_path_factory):
    """Two requests decode for more than two hundred steps: the steps run as recorded graphs while chunks end, windows pass over
    decoded tokens and pages go back to the pool."""
    model = _model("even", tmp_path_factory)
    cfg, _, folder, _ = model
    for dtype in ("float32", "bfloat16"):
        eng = _engine(folder, dtype, cache_tokens=512, max_requests=2)
        a, b = _tokens(cfg, 250, 31), _tokens(cfg, 226, 32)
        schedule = [[("a", 20)], [("b", 3)]] + [[("a", 1), ("b", 1)]] * 216 + [[("a", 14), ("b", 7)]]
        got = zu.run_schedule(eng, {"a": a, "b": b}, schedule)
        assert eng.graph_replays > 150
        assert_logits_close(got["a"], _want(model, a), dtype, f"long decoding a {dtype}")
        assert_logits_close(got["b"], _want(model, b), dtype, f"long decoding b {dtype}")
        eng.cache.check_invariants()


def test_a_slot_and_its_pages_that_are_used_again(tmp_path_factory):
    model = _model("odd", tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, "float32", max_requests=1, cache_tokens=64)
    for seed in (41, 42, 43):
        toks = _tokens(cfg, 40, seed)
        got = zu.run_schedule(eng, {"r": toks}, [[("r", 25)], [("r", 15)]])["r"]
        assert_logits_close(got, _want(model, toks), "float32", f"slot reuse {seed}")


def test_a_fork_carries_chunks_and_windows(tmp_path_factory):
    from glassbox_b200.engine.engine import StepEntry
    model = _model("odd", tmp_path_factory)
    cfg, _, folder, _ = model
    eng = _engine(folder, "float32")
    common, a, b = _tokens(cfg, 37, 91), _tokens(cfg, 16, 92), _tokens(cfg, 16, 93)
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
