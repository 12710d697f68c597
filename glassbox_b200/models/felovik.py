"""Felovik: a decoder with a scaled token embedding and a learned position vector, whose layers norm the residual after the sum
(x <- norm1(alpha x + mixer(x)); x <- norm2(alpha x + ff(x))), whose mixer is a pair side by side on the same input: grouped-query
softmax attention without a rotation (unit-RMS queries and keys, a query temperature that grows with the logarithm of the
position, an output gate per channel) and a selective state-space mixer with one scalar decay per head; each side is normed
over the model width and half their sum is taken. Feed-forwards are a dense clamped gated unit without biases or a mixture of
SwiGLU experts routed by softmax scores within the best groups, the chosen scores renormalised.

This file only *describes* the architecture: which config.json keys it reads and how tensor names map onto part parameters.
The math lives in the parts (``parts/sink_attention.py``, ``parts/state_space.py``, ``parts/parallel.py``, ``parts/mlp.py``,
``parts/moe.py``, ``parts/block.py``, ``parts/embedding.py``).

config.json: ``architecture`` "Felovik"; ``vocab``, ``width``, ``max_positions``; ``norm.eps``; ``embedding.scale``;
``postln_alpha``; ``layers``: a list of {``type``: "parallel", ``mixer``: {``left``: {``heads``, ``kv_heads``, ``dim``, ``vdim``,
``scale``, ``q_temp``: {``coef``, ``every``} (absent: none)}, ``right``: {``heads``, ``groups``, ``vdim``, ``state``, ``conv``,
``norm_groups``}}, ``mlp``: {``kind``: "dense", ``ff``, ``limit``} or {``kind``: "moe", ``expert``: {``ff``}, ``router``: {``experts``,
``top``, ``groups``: {``count``, ``keep``} (absent: none)}} or null}. Tensors of layer i start with ``l<i>.``: ``norm1``, ``norm2``;
``mix.left.q``, ``.k``, ``.v``, ``.g``, ``.o``, ``.out``; ``mix.right.in``, ``.conv``, ``.conv.b``, ``.dt_bias``, ``.A_log``, ``.D``,
``.norm``, ``.o``, ``.out``; dense: ``mlp.gate``, ``mlp.up``, ``mlp.down``; routed: ``mlp.router``, ``mlp.e<j>.gate``, ``.up``,
``.down``; ``embed``, ``pos``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.specs import (ClampedGluSpec, ConfigError, LayerSpec, ModelConfig, ParallelMixerSpec, PositionalEmbeddingSpec, RmsNormSpec,
                            RoutedExpertsSpec, RunSpec, SinkAttentionSpec, StateSpaceSpec)
from ..weights.binding import Ignorable, Stacked

NAME = "Felovik"
#: the slope inside the dense feed-forward's gate activation g * sigmoid(slope * g)
GLU_SLOPE = 1.702
#: what each normed side of the mixer pair weighs in the sum
SIDE_SCALE = 0.5
#: added to the sum of the chosen experts' scores before they are divided by it
RENORM_EPS = 1e-20


def _get(d, key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        raise ConfigError(f"config.json: {where} lacks '{key}'")
    return d[key]


def _pos_int(d, key: str, where: str) -> int:
    v = _get(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"config.json: {where}.{key} must be a positive integer, got {v!r}")
    return v


def _number(d, key: str, where: str) -> float:
    v = _get(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}.{key} must be a number, got {v!r}")
    return float(v)


def _left(m: dict, where: str, eps: float) -> SinkAttentionSpec:
    heads = _pos_int(m, "heads", where)
    kv_heads = _pos_int(m, "kv_heads", where) if "kv_heads" in m else heads
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: heads {heads} is not a multiple of kv_heads {kv_heads}")
    q_temp = None
    if m.get("q_temp") is not None:
        q_temp = (_number(m["q_temp"], "coef", where + ".q_temp"), _number(m["q_temp"], "every", where + ".q_temp"))
        if not q_temp[1] > 0:
            raise ConfigError(f"config.json: {where}.q_temp.every must be positive, got {q_temp[1]!r}")
    return SinkAttentionSpec(num_heads=heads, num_kv_heads=kv_heads, head_dim=_pos_int(m, "dim", where), value_dim=_pos_int(m, "vdim", where),
                             scale=_number(m, "scale", where), window=None, qk_norm_eps=eps, qk_norm_gain=False, q_temp=q_temp,
                             distance_bias=False, sink=False, value_mix="none", output_gate=True, gate_per="channel")


def _right(m: dict, where: str, eps: float) -> StateSpaceSpec:
    heads, vdim = _pos_int(m, "heads", where), _pos_int(m, "vdim", where)
    groups = _pos_int(m, "groups", where) if "groups" in m else 1
    norm_groups = _pos_int(m, "norm_groups", where) if "norm_groups" in m else 1
    if heads % groups:
        raise ConfigError(f"config.json: {where}: heads {heads} is not a multiple of groups {groups}")
    if (heads * vdim) % norm_groups:
        raise ConfigError(f"config.json: {where}: {heads * vdim} channels do not form {norm_groups} equal parts (norm_groups)")
    return StateSpaceSpec(num_heads=heads, num_groups=groups, state_dim=_pos_int(m, "state", where), value_dim=vdim,
                          conv_taps=_pos_int(m, "conv", where), norm_groups=norm_groups, norm_eps=eps)


def _mixer(kind: str, m: dict, where: str, eps: float) -> ParallelMixerSpec:
    if kind != "parallel":
        raise ConfigError(f"config.json: {where}: unknown layer type {kind!r}")
    return ParallelMixerSpec(left=_left(_get(m, "left", where), where + ".left", eps), right=_right(_get(m, "right", where), where + ".right", eps),
                             left_scale=SIDE_SCALE, right_scale=SIDE_SCALE, output_norm=RmsNormSpec(eps=eps), shared_projection=True)


def _feed_forward(mlp, where: str):
    if mlp is None:
        return None
    kind = _get(mlp, "kind", where)
    if kind == "dense":
        limit = _number(mlp, "limit", where)
        if not limit > 0:
            raise ConfigError(f"config.json: {where}.limit must be positive, got {limit!r}")
        return ClampedGluSpec(intermediate_size=_pos_int(mlp, "ff", where), limit=limit, slope=GLU_SLOPE, bias=False)
    if kind == "moe":
        router, expert = _get(mlp, "router", where), _get(mlp, "expert", where)
        experts, top = _pos_int(router, "experts", where + ".router"), _pos_int(router, "top", where + ".router")
        count = keep = 1
        if router.get("groups") is not None:
            w = where + ".router.groups"
            count, keep = _pos_int(router["groups"], "count", w), _pos_int(router["groups"], "keep", w)
            if experts % count or keep > count:
                raise ConfigError(f"config.json: {w}: {experts} experts do not form {count} equal groups of which {keep} are kept")
        if top > keep * (experts // count):
            raise ConfigError(f"config.json: {where}.router: {top} of the {keep * (experts // count)} experts of the kept groups per token")
        return RoutedExpertsSpec(num_experts=experts, top_k=top, expert_size=_pos_int(expert, "ff", where + ".expert"), num_groups=count,
                                 keep_groups=keep, correction=False, shared_size=0, shared_gate=False, scoring="softmax",
                                 group_score="best", renormalise=RENORM_EPS, activation="swiglu")
    raise ConfigError(f"config.json: {where}: unknown kind {kind!r}")


def parse_felovik_config(raw: dict) -> ModelConfig:
    vocab = _pos_int(raw, "vocab", "top level")
    width = _pos_int(raw, "width", "top level")
    max_pos = _pos_int(raw, "max_positions", "top level")
    eps = _number(_get(raw, "norm", "top level"), "eps", "norm")
    if not eps > 0:
        raise ConfigError(f"config.json: norm.eps must be positive, got {eps!r}")
    alpha = _number(raw, "postln_alpha", "top level")
    scale = _number(_get(raw, "embedding", "top level"), "scale", "embedding")
    layers_raw = _get(raw, "layers", "top level")
    if not isinstance(layers_raw, list) or not layers_raw:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    norm = RmsNormSpec(eps=eps)
    layers, schedule = [], []
    for i, L in enumerate(layers_raw):
        where = f"layers[{i}]"
        mixer = _mixer(_get(L, "type", where), _get(L, "mixer", where), where + ".mixer", eps)
        ffn = _feed_forward(L.get("mlp"), where + ".mlp")
        layers.append(LayerSpec(mixer=mixer, ffn=ffn, mixer_norm=None, ffn_norm=None, arrangement="post_norm", mixer_post_norm=norm,
                                ffn_post_norm=norm if ffn is not None else None, residual_scale=alpha))
        schedule.append(RunSpec(layer=i, cache=i))
    return ModelConfig(architecture=NAME, vocab_size=vocab, hidden_size=width, max_position=max_pos, tie_word_embeddings=False,
                       layers=tuple(layers), schedule=tuple(schedule), final_norm=norm, raw=dict(raw),
                       embedding=PositionalEmbeddingSpec(max_position=max_pos, scale=scale))


def bind_felovik_weights(config: ModelConfig) -> dict:
    b = {"embed.weight": Stacked(("embed",)), "embed.positions": Stacked(("pos",)), "final_norm.weight": Stacked(("final.norm",)),
         "head.weight": Stacked(("head",))}
    unused = []
    for i, layer in enumerate(config.layers):
        p, t = f"layers.{i}", f"l{i}"
        lf, rt = f"{t}.mix.left", f"{t}.mix.right"
        b[f"{p}.mixer_post_norm.weight"] = Stacked((f"{t}.norm1",))
        b[f"{p}.mixer.w_in"] = Stacked((f"{lf}.q", f"{lf}.k", f"{lf}.v", f"{lf}.g", f"{rt}.in"))
        b[f"{p}.mixer.left.wo"] = Stacked((f"{lf}.o",))
        b[f"{p}.mixer.left_norm.weight"] = Stacked((f"{lf}.out",))
        b[f"{p}.mixer.right.conv"] = Stacked((f"{rt}.conv",))
        b[f"{p}.mixer.right.conv_bias"] = Stacked((f"{rt}.conv.b",))
        b[f"{p}.mixer.right.dt_bias"] = Stacked((f"{rt}.dt_bias",))
        b[f"{p}.mixer.right.a_log"] = Stacked((f"{rt}.A_log",))
        b[f"{p}.mixer.right.skip"] = Stacked((f"{rt}.D",))
        b[f"{p}.mixer.right.out_norm"] = Stacked((f"{rt}.norm",))
        b[f"{p}.mixer.right.wo"] = Stacked((f"{rt}.o",))
        b[f"{p}.mixer.right_norm.weight"] = Stacked((f"{rt}.out",))
        if layer.ffn is None:
            unused.append(f"{t}.norm2")         # a file may store it for every layer
            continue
        f = f"{t}.mlp"
        b[f"{p}.ffn_post_norm.weight"] = Stacked((f"{t}.norm2",))
        if isinstance(layer.ffn, ClampedGluSpec):
            b[f"{p}.ffn.w_gate_up"] = Stacked((f"{f}.gate", f"{f}.up"))
            b[f"{p}.ffn.w_down"] = Stacked((f"{f}.down",))
        else:
            E = layer.ffn.num_experts
            b[f"{p}.ffn.router"] = Stacked((f"{f}.router",))
            b[f"{p}.ffn.w_up"] = Stacked(tuple(f"{f}.e{j}.{which}" for j in range(E) for which in ("gate", "up")))
            b[f"{p}.ffn.w_down"] = Stacked(tuple(f"{f}.e{j}.down" for j in range(E)))
    if unused:
        b[Ignorable.KEY] = Ignorable(tuple(unused))
    return b


def make_felovik_raw_config(*, vocab: int, width: int, max_positions: int, layers: list, alpha: float, embedding_scale: float = 1.0,
                            norm_eps: float = 1e-6) -> dict:
    """``layers``: a list of dicts as config.json holds them ({"type", "mixer", "mlp"})."""
    return {"architecture": NAME, "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": norm_eps},
            "embedding": {"scale": embedding_scale}, "postln_alpha": alpha, "layers": layers}


register_architecture(Architecture(name=NAME, parse=parse_felovik_config, bind=bind_felovik_weights, make_raw_config=make_felovik_raw_config),
                      replace=True)
