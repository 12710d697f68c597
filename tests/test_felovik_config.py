"""Felovik without a GPU: the configuration reader (every optional key present and absent, every refusal), the binding of
tensor names to parameters, and properties of the plain implementation that the GPU tests compare against."""
import math

import numpy as np
import pytest

import glassbox_b200  # noqa: F401  (registers the architectures)
from glassbox_b200.config.registry import get_architecture, parse_config
from glassbox_b200.config.specs import (ClampedGluSpec, ConfigError, ParallelMixerSpec, PositionalEmbeddingSpec, RmsNormSpec, RoutedExpertsSpec,
                                        SinkAttentionSpec, StateSpaceSpec)
from glassbox_b200.engine.model import DecoderModel
from glassbox_b200.parts.base import CombinedCacheSpec, PagedKvSpec, StateSpec, build_part
from glassbox_b200.weights.binding import Ignorable
from plain import felovik_plain as plain
import felovik_util as fu


@pytest.mark.parametrize("name", sorted(fu.CONFIGS))
def test_every_tensor_is_bound(name):
    raw = fu.CONFIGS[name]()
    config = parse_config(raw)
    model = DecoderModel(config)
    specs, binding = model.param_specs(), get_architecture("Felovik").bind(config)
    unused = binding.pop(Ignorable.KEY, Ignorable(()))
    assert set(unused.names) == {f"l{i}.norm2" for i, L in enumerate(raw["layers"]) if L["mlp"] is None}
    assert set(binding) == set(specs)
    shapes = fu.tensor_shapes(raw)
    assert sorted(n for path in specs for n in binding[path].names) == sorted(shapes)
    for path, spec in specs.items():
        names = binding[path].names
        rows = spec.pieces if len(names) > 1 else ((spec.shape[0],) if spec.shape else ())
        for n, r in zip(names, rows):
            assert tuple(shapes[n]) == (r,) + tuple(spec.shape[1:]), n


def test_what_the_reader_makes_of_the_keys():
    config = parse_config(fu.CONFIGS["odd"]())
    assert config.vocab_size == 203 and config.hidden_size == 56 and config.max_position == 512 and config.residual_streams == 0
    assert config.embedding == PositionalEmbeddingSpec(max_position=512, scale=2.5)
    norm = RmsNormSpec(eps=1e-5)
    assert config.final_norm == norm
    assert all(l.arrangement == "post_norm" and l.residual_scale == 1.7 and l.mixer_post_norm == norm and l.mixer_norm is None
               for l in config.layers)
    a, b, c, d = config.layers
    assert isinstance(a.mixer, ParallelMixerSpec) and (a.mixer.left_scale, a.mixer.right_scale) == (0.5, 0.5)
    assert a.mixer.output_norm == norm and a.mixer.shared_projection
    assert a.mixer.left == SinkAttentionSpec(num_heads=6, num_kv_heads=2, head_dim=20, value_dim=12, scale=20 ** -0.5, window=None,
                                             qk_norm_eps=1e-5, qk_norm_gain=False, q_temp=(0.4, 7.0), distance_bias=False, sink=False,
                                             value_mix="none", output_gate=True, gate_per="channel")
    assert a.mixer.right == StateSpaceSpec(num_heads=4, num_groups=2, state_dim=12, value_dim=6, conv_taps=4, norm_groups=3, norm_eps=1e-5)
    assert a.ffn == ClampedGluSpec(intermediate_size=40, limit=0.8, slope=1.702, bias=False)
    assert b.ffn == RoutedExpertsSpec(num_experts=6, top_k=2, expert_size=24, num_groups=3, keep_groups=2, correction=False, shared_size=0,
                                      shared_gate=False, scoring="softmax", group_score="best", renormalise=1e-20, activation="swiglu")
    assert c.ffn is None and c.ffn_post_norm is None and c.mixer.left.q_temp is None
    assert d.ffn.num_groups == 1 and d.ffn.keep_groups == 1
    specs = DecoderModel(config).cache_layer_specs()
    # S, then a ring of as many inputs as there are taps
    assert specs[0] == CombinedCacheSpec(PagedKvSpec(2, 20, None, value_dim=12), (("right", StateSpec((4 * 12 * 6 + 4 * (24 + 2 * 2 * 12),))),))
    # (rounded up to whole 16-byte pieces)
    assert specs[2] == CombinedCacheSpec(PagedKvSpec(4, 12, None, value_dim=8), (("right", StateSpec((2 * 10 * 14 + 3 * (28 + 2 * 10),))),))


def test_one_projection_serves_both_sides():
    config = parse_config(fu.CONFIGS["odd"]())
    specs = DecoderModel(config).param_specs()
    assert "layers.0.mixer.w_in" in specs and not any(p.endswith(("left.w_in", "right.w_in")) for p in specs)
    left_cols = (6 + 2) * 20 + 2 * 12 + 6 * 12
    right_cols = 24 + 24 + 2 * 2 * 12 + 4
    assert specs["layers.0.mixer.w_in"].shape == (left_cols + right_cols, 56)
    # the same mixers on their own have projections of their own
    lone = build_part("mixer", config.layers[0].mixer.right, hidden_size=56)
    assert lone.param_specs()["w_in"].shape == (right_cols, 56)


def _broken(change):
    raw = fu.CONFIGS["odd"]()
    change(raw)
    return raw


@pytest.mark.parametrize("change, word", [
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r.pop("max_positions"), "max_positions"),
    (lambda r: r.pop("postln_alpha"), "postln_alpha"),
    (lambda r: r["embedding"].pop("scale"), "scale"),
    (lambda r: r["norm"].__setitem__("eps", 0.0), "eps"),
    (lambda r: r["layers"][0].__setitem__("type", "conv"), "unknown layer type"),
    (lambda r: r["layers"][0]["mixer"].pop("right"), "right"),
    (lambda r: r["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 4), "multiple"),
    (lambda r: r["layers"][0]["mixer"]["left"]["q_temp"].pop("coef"), "coef"),
    (lambda r: r["layers"][0]["mixer"]["left"]["q_temp"].__setitem__("every", 0), "every"),
    (lambda r: r["layers"][0]["mixer"]["right"].__setitem__("groups", 3), "multiple"),
    (lambda r: r["layers"][0]["mixer"]["right"].__setitem__("norm_groups", 5), "norm_groups"),
    (lambda r: r["layers"][0]["mixer"]["right"].pop("conv"), "conv"),
    (lambda r: r["layers"][0]["mlp"].__setitem__("kind", "sparse"), "unknown kind"),
    (lambda r: r["layers"][0]["mlp"].__setitem__("limit", -1.0), "limit"),
    (lambda r: r["layers"][1]["mlp"]["router"].__setitem__("top", 5), "experts of the kept groups"),
    (lambda r: r["layers"][1]["mlp"]["router"]["groups"].__setitem__("count", 4), "equal groups"),
    (lambda r: r["layers"][1]["mlp"]["router"]["groups"].__setitem__("keep", 4), "kept"),
    (lambda r: r.__setitem__("layers", []), "layers"),
])
def test_refusals_name_the_key(change, word):
    with pytest.raises(ConfigError) as e:
        parse_config(_broken(change))
    assert word in str(e.value)


# ----------------------------------------------------------------------------- the plain implementation's own equations
def test_query_temperature_steps():
    t = {"coef": 0.5, "every": 4}
    values = [plain.query_temperature(p, t) for p in range(12)]
    assert values[:3] == [1.0] * 3 and values[3] == values[6] == pytest.approx(1 + 0.5 * math.log(2))
    assert values[7] == values[10] == pytest.approx(1 + 0.5 * math.log(3)) and values[11] == pytest.approx(1 + 0.5 * math.log(4))
    assert plain.query_temperature(1000, None) == 1.0
    assert plain.query_temperature(0, {"coef": 0.5, "every": 1}) == pytest.approx(1 + 0.5 * math.log(2))


def test_the_state_keeps_everything_without_decay_and_nothing_under_a_strong_one():
    rng = np.random.default_rng(0)
    T, H, V, G, N = 6, 2, 3, 1, 4
    x, B, C = rng.standard_normal((T, H, V)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt = rng.uniform(0.5, 1.5, (T, H))
    D = np.array([0.0, 2.0])
    y = plain.ssd_scan(x, B, C, dt, np.array([-60.0, 60.0]), D)
    for t in range(T):
        kept = sum(dt[j, 0] * (B[j, 0] @ C[t, 0]) * x[j, 0] for j in range(t + 1))
        assert np.allclose(y[t, 0], kept)
        assert np.allclose(y[t, 1], dt[t, 1] * (B[t, 0] @ C[t, 0]) * x[t, 1] + 2.0 * x[t, 1])


def test_portions_continue_from_the_state_in_chunked_form():
    """The recurrence equals its chunked form: inside a chunk by decay ratios, from the chunk's start by the state."""
    rng = np.random.default_rng(1)
    T, V, N, L = 11, 2, 3, 4
    x, B, C = rng.standard_normal((T, 1, V)), rng.standard_normal((T, 1, N)), rng.standard_normal((T, 1, N))
    dt, a_log = rng.uniform(0.1, 1.0, (T, 1)), np.array([0.3])
    want = plain.ssd_scan(x, B, C, dt, a_log, np.array([0.7]))
    S = np.zeros((N, V))
    for c0 in range(0, T, L):
        rows = range(c0, min(c0 + L, T))
        cum = np.cumsum([-math.exp(a_log[0]) * dt[t, 0] for t in rows])
        for i, t in enumerate(rows):
            y = math.exp(cum[i]) * (S.T @ C[t, 0]) + 0.7 * x[t, 0]
            y = y + sum(math.exp(cum[i] - cum[j]) * dt[c0 + j, 0] * (B[c0 + j, 0] @ C[t, 0]) * x[c0 + j, 0] for j in range(i + 1))
            assert np.allclose(y, want[t, 0])
        S = math.exp(cum[-1]) * S + sum(math.exp(cum[-1] - cum[j]) * dt[t, 0] * np.outer(B[t, 0], x[t, 0]) for j, t in enumerate(rows))


def test_groups_score_by_their_best_and_the_rest_cannot_be_chosen():
    s = [0.30, 0.01, 0.20, 0.19, 0.02, 0.28]
    assert plain.choose(s, 2, 3, 2) == [0, 5]                  # runs {0,1}, {2,3}, {4,5}: best 0.30, 0.20, 0.28
    assert plain.choose(s, 3, 3, 2) == [0, 5, 4]               # (2 and 3 are larger than 4, but their run is not kept)
    assert plain.choose(s, 3, 1, 1) == [0, 5, 2]
    W = {"router": np.log(np.array(s))[:, None]}
    order, weight = plain.route(np.array([[1.0]]), W, "", {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}})
    assert list(order[0]) == [0, 5] and np.allclose(weight[0], [0.30 / 0.58, 0.28 / 0.58])


def test_the_gate_comes_before_the_norm_and_parts_are_normed_apart():
    rng = np.random.default_rng(2)
    y, z, w = rng.standard_normal((3, 12)), rng.standard_normal((3, 12)), rng.standard_normal(12)
    out = plain.grouped_gated_norm(y, z, w, 3, 1e-12)
    u = y * plain.silu(z)
    for g in range(3):
        part = u[:, 4 * g:4 * g + 4]
        assert np.allclose(out[:, 4 * g:4 * g + 4], part / np.sqrt((part ** 2).mean(1, keepdims=True)) * w[4 * g:4 * g + 4])
    y2 = y.copy()
    y2[:, :4] *= 7.0                                           # a part's size is normed away and touches no other part
    assert np.allclose(plain.grouped_gated_norm(y2, z, w, 3, 1e-12), out)


def test_convolution_with_a_bias_starts_from_zeros():
    x = np.arange(12.0).reshape(6, 2)
    y = plain.causal_conv(x, np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]]), np.array([0.5, -1.0]))
    assert np.array_equal(y[:, 1], x[:, 1] - 1.0) and y[0, 0] == 0.5 and y[2, 0] == 10.0 * 2 + 100.0 * 4 + 0.5


def test_the_clamps_of_the_dense_unit():
    W = {"gate": np.array([[1.0]]), "up": np.array([[1.0]]), "down": np.array([[1.0]])}
    f = lambda v: float(plain.dense_ff(np.array([[v]]), W, "", {"limit": 1.5})[0, 0])
    assert f(9.0) == pytest.approx(1.5 / (1 + math.exp(-1.702 * 1.5)) * 2.5)
    assert f(-9.0) == pytest.approx(-9.0 / (1 + math.exp(1.702 * 9.0)) * -0.5)           # the gate is cut from above only
