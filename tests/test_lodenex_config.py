"""Lodenex without a GPU: the configuration reader (every optional key present and absent, every refusal), the binding of
tensor names to parameters, the frequencies of both rotations, and properties of the plain implementation that the GPU tests
compare against."""
import math

import numpy as np
import pytest

import glassbox_b200  # noqa: F401  (registers the architectures)
from glassbox_b200.config.registry import get_architecture, parse_config
from glassbox_b200.config.specs import (CappedLmHeadSpec, ConfigError, GeluMlpSpec, LatentAttentionSpec, LmHeadSpec, RmsNormSpec,
                                        RopeBandRescaleSpec, RopeRescaleSpec, RopeSpec, ScaledEmbeddingSpec, SinkAttentionSpec)
from glassbox_b200.engine.model import DecoderModel
from glassbox_b200.kernels import latent_decode_splits
from glassbox_b200.parts.base import PagedKvSpec, build_part
from glassbox_b200.parts.rope import inverse_frequencies, rescaled_frequencies
from plain import lodenex_plain as plain
import lodenex_util as lu


@pytest.mark.parametrize("name", sorted(lu.CONFIGS))
def test_every_tensor_is_bound(name):
    raw = lu.CONFIGS[name]()
    config = parse_config(raw)
    specs, binding = DecoderModel(config).param_specs(), get_architecture("Lodenex").bind(config)
    assert set(binding) == set(specs)
    shapes = lu.tensor_shapes(raw)
    assert sorted(n for path in specs for n in binding[path].names) == sorted(shapes)
    for path, spec in specs.items():
        names = binding[path].names
        rows = spec.pieces if len(names) > 1 else (spec.shape[0],)
        for n, r in zip(names, rows):
            assert tuple(shapes[n]) == (r,) + tuple(spec.shape[1:]), n


def test_what_the_reader_makes_of_the_keys():
    config = parse_config(lu.CONFIGS["odd"]())
    assert config.vocab_size == 203 and config.hidden_size == 56 and config.residual_streams == 0
    assert config.embedding == ScaledEmbeddingSpec(scale=2.5) and config.head == CappedLmHeadSpec(softcap=6.0)
    norm = RmsNormSpec(eps=1e-5)
    assert config.final_norm == norm
    assert all(l.arrangement == "branch_norm" and l.mixer_post_norm == norm and l.mixer_norm is None for l in config.layers)
    a, b, c, d, e, f = config.layers
    top = config.max_position
    assert a.mixer == SinkAttentionSpec(
        num_heads=6, num_kv_heads=2, head_dim=20, value_dim=12, scale=1.5 * 20 ** -0.5, chunk=23, softcap=3.0, qk_norm_eps=1e-5,
        qk_norm_over="projection", distance_bias=False, sink=True, output_gate=True, gate_per="head",
        position=RopeSpec(theta=10000.0, rotary_dim=12, max_position=top, pairing="half", rescale=RopeBandRescaleSpec(5.0, 40.0, 1.0, 3.0)))
    assert b.mixer == LatentAttentionSpec(
        num_heads=3, nope_dim=10, rope_dim=6, value_dim=12, latent_dim=22, scale=1.5 * 16 ** -0.5, latent_eps=1e-5, sink=False, window=13,
        q_rank=18, output_gate=True,
        position=RopeSpec(theta=10000.0, rotary_dim=6, max_position=top, pairing="half", rescale=RopeRescaleSpec(3.0, 64.0, 8.0, 1.0)))
    assert a.ffn == GeluMlpSpec(intermediate_size=40) and c.ffn is None and c.ffn_post_norm is None
    assert c.mixer.chunk is None and c.mixer.softcap is None and c.mixer.position.rescale is None
    assert d.mixer.window is None and d.mixer.position.rescale is None and e.mixer.position.theta == 500.0
    assert parse_config(lu.CONFIGS["ragged"]()).head == LmHeadSpec()
    specs = DecoderModel(config).cache_layer_specs()
    assert specs[0] == PagedKvSpec(2, 20, None, value_dim=12, chunk=23) and specs[2] == PagedKvSpec(1, 10, None, value_dim=24)
    assert specs[1] == PagedKvSpec(1, 28, 13, value_dim=0) and specs[3] == PagedKvSpec(1, 22, None, value_dim=0)


def test_the_query_rank_is_read_off_the_tensors_where_no_key_has_it():
    raw = lu.CONFIGS["odd"]()
    shapes = lu.tensor_shapes(raw)
    ranks = [L["mixer"].pop("q_rank") for L in raw["layers"] if "q_rank" in L["mixer"]]
    config = parse_config(raw, shapes)
    assert [l.mixer.q_rank for l in config.layers if isinstance(l.mixer, LatentAttentionSpec)] == ranks
    with pytest.raises(ConfigError, match="q_rank"):
        parse_config(raw)


def _broken(change):
    raw = lu.CONFIGS["odd"]()
    change(raw)
    return raw


def _m(i, key, value):
    return lambda r: r["layers"][i]["mixer"].__setitem__(key, value)


@pytest.mark.parametrize("change, word", [
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r["embedding"].pop("scale"), "scale"),
    (lambda r: r["norm"].__setitem__("eps", 0.0), "eps"),
    (lambda r: r.__setitem__("logit_softcap", -1.0), "logit_softcap"),
    (lambda r: r.__setitem__("layers", []), "layers"),
    (lambda r: r["layers"][0].__setitem__("type", "conv"), "unknown layer type"),
    (_m(0, "kv_heads", 4), "multiple"),
    (_m(0, "softcap", 0), "softcap"),
    (_m(0, "mask", {"size": 0}), "size"),
    (lambda r: r["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda r: r["layers"][0]["mixer"]["rot"].__setitem__("dims", 22), "at most 20"),
    (lambda r: r["layers"][0]["mixer"]["rot"].__setitem__("dims", 7), "even"),
    (lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].pop("high"), "high"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].__setitem__("factor", 0.0), "factor"),
    (lambda r: r["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (_m(1, "mask", {}), "size"),
    (lambda r: r["layers"][0]["mlp"].__setitem__("kind", "sparse"), "unknown kind"),
    (lambda r: r["layers"][0]["mlp"].__setitem__("ff", 0), "ff"),
])
def test_refusals_name_the_key(change, word):
    with pytest.raises(ConfigError) as e:
        parse_config(_broken(change))
    assert word in str(e.value)


def test_what_the_parts_refuse():
    rope = RopeSpec(theta=100.0, rotary_dim=8, max_position=64)
    attn = dict(num_heads=2, num_kv_heads=1, head_dim=8, value_dim=8, scale=1.0, distance_bias=False)
    for kw, word in ((dict(chunk=4, window=4), "chunk"), (dict(chunk=0), "chunk"), (dict(softcap=-1.0), "softcap"),
                     (dict(position=rope, qk_norm_over="projection", value_mix="source"), "value mix"),
                     (dict(position=rope, qk_norm_eps=1e-6), "per head"), (dict(qk_norm_over="row"), "qk_norm_over"),
                     (dict(position=RopeSpec(theta=100.0, rotary_dim=8, max_position=64, pairing="interleaved")), "half"),
                     (dict(position=RopeSpec(theta=100.0, rotary_dim=10, max_position=64)), "do not fit")):
        with pytest.raises(ValueError, match=word):
            build_part("mixer", SinkAttentionSpec(**attn, **kw), hidden_size=16)
    lat = dict(num_heads=2, nope_dim=4, rope_dim=8, value_dim=4, latent_dim=6, scale=1.0, latent_eps=1e-6)
    with pytest.raises(ValueError, match="half"):
        build_part("mixer", LatentAttentionSpec(**lat, q_rank=4, position=RopeSpec(theta=9.0, rotary_dim=8, max_position=8, pairing="interleaved")),
                   hidden_size=16)
    # a gate without a query latent, and a query latent over another layer's cache, are each fine
    p = build_part("mixer", LatentAttentionSpec(**lat, position=rope, output_gate=True), hidden_size=16)
    assert p.param_specs()["w_in"].pieces == (24, 14, 8)
    p = build_part("mixer", LatentAttentionSpec(**lat, position=rope, output_gate=True, q_rank=5, kv_source=0), hidden_size=16)
    assert p.param_specs()["w_in"].pieces == (5, 8) and "latent_norm" not in p.param_specs()


@pytest.mark.parametrize("dims, base, sc", [
    (40, 10000.0, lu.bands(6.0, 1000, 1.0, 5.0)), (12, 500.0, lu.bands(3.0, 40, 1.0, 3.0)), (64, 1e6, lu.bands(32.0, 8192, 1.0, 4.0)),
    (2, 10.0, lu.bands(2.0, 10, 0.5, 2.0)), (20, 10000.0, lu.bands(4.0, 100000000, 1.0, 4.0)), (20, 10000.0, lu.bands(4.0, 1, 1.0, 4.0)), (6, 10.0, None)])
def test_frequencies_in_bands(dims, base, sc):
    rescale = RopeBandRescaleSpec(sc["factor"], sc["original"], sc["low"], sc["high"]) if sc else None
    got, length = rescaled_frequencies(base, dims, rescale)
    want, one = plain.frequencies_by_wavelength(dims, base, sc)
    np.testing.assert_allclose(got, want, rtol=1e-12)
    assert length == one == 1.0
    np.testing.assert_allclose(inverse_frequencies(base, dims, rescale).numpy(), np.array(want, dtype=np.float32), rtol=1e-7)


def test_the_three_bands_of_frequencies():
    """Wavelengths below, between and above the two edges: kept, mixed in proportion, divided."""
    f = plain.base_frequencies(8, 10000.0)                       # wavelengths 2 pi x (1, 10, 100, 1000)
    got, _ = plain.frequencies_by_wavelength(8, 10000.0, lu.bands(4.0, 2 * math.pi * 200, 1.0, 4.0))      # edges at 2 pi x 50 and 2 pi x 200
    assert got[:2] == f[:2] and got[3] == f[3] / 4
    s = (2.0 - 1.0) / 3.0
    assert got[2] == pytest.approx((1 - s) * f[2] / 4 + s * f[2])
    got, _ = plain.frequencies_by_wavelength(8, 10000.0, lu.bands(4.0, 2 * math.pi * 100, 1.0, 4.0))      # exactly at the long edge
    assert got[2] == pytest.approx(f[2] / 4)


@pytest.mark.parametrize("dims, base, sc", [
    (24, 10000.0, lu.ramp(5.0, 2000, 32.0, 1.0)), (10, 300.0, lu.ramp(2.0, 200, 16.0, 2.0)), (64, 1e6, lu.ramp(40.0, 4096, 32.0, 1.0)),
    (2, 10.0, lu.ramp(3.0, 8, 4.0, 1.0)), (8, 10000.0, lu.ramp(3.0, 4, 32.0, 1.0)), (8, 50.0, None)])
def test_frequencies_along_a_ramp(dims, base, sc):
    rescale = RopeRescaleSpec(sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc else None
    got, length = rescaled_frequencies(base, dims, rescale)
    want, longer = plain.frequencies_by_turns(dims, base, sc)
    np.testing.assert_allclose(got, want, rtol=1e-12)
    assert length == pytest.approx(longer) and longer == pytest.approx(1.0 if sc is None else 1.0 + 0.1 * math.log(sc["factor"]))


def test_shares_of_a_latent_decode_cover_the_tiles_without_idle_ones():
    for heads in (1, 4, 16, 17, 32, 128):
        for seqs in (1, 2, 7, 8, 16, 33, 64, 300):
            for keys in (1, 64, 65, 1000, 1024, 4096, 100000):
                tiles, s = -(-keys // 64), latent_decode_splits(seqs, heads, keys)
                assert 1 <= s <= 64 and s <= tiles
                assert -(-tiles // -(-tiles // s)) == s, (heads, seqs, keys, s)
    assert latent_decode_splits(64, 16, 1024) < latent_decode_splits(8, 16, 1024)


# ----------------------------------------------------------------------------- the plain implementation's own equations
def test_chunks_and_windows_by_hand():
    assert plain.chunk_keys(0, 4) == [0] and plain.chunk_keys(3, 4) == [0, 1, 2, 3] and plain.chunk_keys(4, 4) == [4]
    assert plain.chunk_keys(6, 4) == [4, 5, 6] and plain.chunk_keys(5, 1) == [5] and plain.chunk_keys(2, None) == [0, 1, 2]
    assert plain.window_keys(6, 4) == [3, 4, 5, 6] and plain.window_keys(2, 4) == [0, 1, 2] and plain.window_keys(5, 1) == [5]


def test_a_sink_takes_its_share_and_is_neither_scaled_nor_capped():
    w = plain.sink_softmax(np.zeros(3), math.log(5.0))
    assert np.allclose(w, 1 / 8)
    assert np.allclose(plain.sink_softmax(np.array([1.0, 2.0]), None).sum(), 1.0)
    q, k, v = np.ones((1, 1, 1)), np.full((1, 1, 1), 100.0), np.ones((1, 1, 1))
    out = plain.capped_attention(q, k, v, 1.0, 2.0, np.array([7.0]), 4)        # the score is capped to 2, the sink stays 7
    assert out[0, 0, 0] == pytest.approx(math.exp(2.0) / (math.exp(2.0) + math.exp(7.0)))


def test_the_exact_gelu():
    assert plain.gelu(0.0) == 0.0 and plain.gelu(1.0) == pytest.approx(0.8413447460685429) and plain.gelu(-1.0) == pytest.approx(-0.15865525393145707)
    assert plain.gelu(np.array([8.0])) == pytest.approx(8.0)


def test_rotation_keeps_lengths_and_depends_on_differences():
    rng = np.random.default_rng(0)
    freqs, length = plain.frequencies_by_turns(6, 50.0, lu.ramp(3.0, 30, 4.0, 1.0))
    q, k = rng.standard_normal(9), rng.standard_normal(9)
    a = plain.rotate(q, 11, freqs, length) @ plain.rotate(k, 4, freqs, length)
    b = plain.rotate(q, 27, freqs, length) @ plain.rotate(k, 20, freqs, length)
    assert a == pytest.approx(b)
    assert np.array_equal(plain.rotate(q, 5, freqs, length)[6:], q[6:])          # the rest passes unchanged
    turned = plain.rotate(q, 5, freqs, length)
    assert np.hypot(turned[1], turned[4]) == pytest.approx(length * np.hypot(q[1], q[4]))   # component 1 turns with component 4


def test_queries_are_normed_over_all_heads_at_once():
    rng = np.random.default_rng(1)
    m = lu.attention(2, 1, 4, 4, 2, chunk=8)
    W = {"q": rng.standard_normal((8, 5)), "k": rng.standard_normal((4, 5)), "v": rng.standard_normal((4, 5)), "g": rng.standard_normal((2, 5)),
         "o": np.eye(8), "q.norm": np.ones(8), "k.norm": np.ones(4), "sink": np.zeros(2)}
    h = rng.standard_normal((6, 5))
    base = plain.attention(h, W, "", m, 1e-12)
    scaled = dict(W, q=W["q"] * 3.0)
    assert np.allclose(plain.attention(h, scaled, "", m, 1e-12), base)          # a factor on all heads is normed away
    one = W["q"].copy()
    one[:4] *= 3.0                                                               # on one head it changes the other as well
    got = plain.attention(h, dict(W, q=one), "", m, 1e-12)
    assert not np.allclose(got[:, 4:], base[:, 4:])
