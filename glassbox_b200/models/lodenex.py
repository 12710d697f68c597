"""Lodenex: a decoder with a scaled token embedding whose layers norm their branches on the way out only (x += norm1(mixer(x));
x += norm2(ff(x)), the branches reading the residual itself), whose mixers are either grouped-query softmax attention within
chunks of positions (queries and keys RMS-normed over their whole projections and rotated with frequencies stretched in bands
of wavelength, capped scores, a learned sink logit per head, a sigmoid gate per head) or attention over a compressed latent
cache within a sliding window (queries through a latent of their own, a rotated part with frequencies stretched along a ramp
over the pairs, a sigmoid gate per output channel), whose feed-forwards are dense with the exact GELU, and whose logits are
capped.

This file only *describes* the architecture: which config.json keys it reads and how tensor names map onto part parameters.
The math lives in the parts (``parts/sink_attention.py``, ``parts/latent_attention.py``, ``parts/rope.py``, ``parts/mlp.py``,
``parts/block.py``, ``parts/embedding.py``).

config.json: ``architecture`` "Lodenex"; ``vocab``, ``width``; ``norm.eps``; ``embedding.scale``; ``logit_softcap``; ``layers``: a
list of {``type``: "attention", ``mixer``: {``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap``, ``mask.size``,
``rot``: {``base``, ``dims``, ``scaling``: {``factor``, ``low``, ``high``, ``original``}}}} or {``type``: "latent_attention",
``mixer``: {``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``q_rank``, ``scale``, ``mask.size``, ``rot``: {``base``, ``dims``,
``scaling``: {``factor``, ``original``, ``fast``, ``slow``}}}}, each with ``mlp``: {``kind``: "dense", ``ff``} or null. Absent: ``softcap``
and ``logit_softcap`` (no cap), ``mask`` (every earlier token is visible), ``scaling`` (plain frequencies), ``q_rank`` (read off
the tensors). Tensors of layer i start with ``l<i>.``: ``norm1``, ``norm2``; attention: ``mix.q``, ``.k``, ``.v``, ``.g``, ``.o``,
``.q.norm``, ``.k.norm``, ``.sink``; latent attention: ``mix.dq``, ``.dq.norm``, ``.uq``, ``.dkv``, ``.dkv.norm``, ``.uk``, ``.uv``, ``.g``,
``.o``; ``mlp.up``, ``mlp.down``; ``embed``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import Dict, Optional

from ..config.registry import Architecture, register_architecture
from ..config.specs import (CappedLmHeadSpec, ConfigError, GeluMlpSpec, LatentAttentionSpec, LayerSpec, LmHeadSpec, ModelConfig,
                            RmsNormSpec, RopeBandRescaleSpec, RopeRescaleSpec, RopeSpec, RunSpec, ScaledEmbeddingSpec,
                            SinkAttentionSpec)
from ..weights.binding import Stacked

NAME = "Lodenex"
#: no key limits the length of a sequence; angles are formed on the device, so this only bounds requests
DEFAULT_MAX_POSITION = 1 << 20


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


def _positive(d, key: str, where: str) -> float:
    v = _number(d, key, where)
    if not v > 0:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {v!r}")
    return v


def _cap(d: dict, key: str, where: str) -> Optional[float]:
    return _positive(d, key, where) if d.get(key) is not None else None


def _rotation(m: dict, where: str, largest: int, max_pos: int, rescale_kind) -> RopeSpec:
    """The rotation of the first ``rot.dims`` channels; the frequencies of an "attention" layer are stretched in bands, those of a
    "latent_attention" layer along a ramp (``rescale_kind``)."""
    rot, w = _get(m, "rot", where), where + ".rot"
    dims = _pos_int(rot, "dims", w)
    if dims % 2 or dims > largest:
        raise ConfigError(f"config.json: {w}.dims {dims} must be even and at most {largest}")
    rescale, sc = None, rot.get("scaling")
    if sc is not None:
        w += ".scaling"
        if rescale_kind is RopeBandRescaleSpec:
            rescale = RopeBandRescaleSpec(factor=_positive(sc, "factor", w), original=_positive(sc, "original", w),
                                          low=_positive(sc, "low", w), high=_positive(sc, "high", w))
        else:
            rescale = RopeRescaleSpec(factor=_positive(sc, "factor", w), original=_positive(sc, "original", w),
                                      fast=_positive(sc, "fast", w), slow=_positive(sc, "slow", w))
    return RopeSpec(theta=_positive(rot, "base", where + ".rot"), rotary_dim=dims, max_position=max_pos, pairing="half", rescale=rescale)


def _q_rank(m: dict, tensor: str, shapes: Optional[Dict[str, tuple]], where: str) -> int:
    if m.get("q_rank") is not None:
        return _pos_int(m, "q_rank", where)
    if shapes is not None and len(shapes.get(tensor, ())) == 2:
        return int(shapes[tensor][0])
    raise ConfigError(f"config.json: {where}: the rank 'q_rank' is neither given nor readable from the shape of {tensor}")


def _mixer(kind: str, m: dict, i: int, where: str, eps: float, max_pos: int, shapes):
    size = _pos_int(m["mask"], "size", where + ".mask") if m.get("mask") is not None else None
    heads = _pos_int(m, "heads", where)
    if kind == "attention":
        kv_heads, dim = _pos_int(m, "kv_heads", where), _pos_int(m, "dim", where)
        if heads % kv_heads:
            raise ConfigError(f"config.json: {where}: heads {heads} is not a multiple of kv_heads {kv_heads}")
        return SinkAttentionSpec(num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, value_dim=_pos_int(m, "vdim", where),
                                 scale=_number(m, "scale", where), chunk=size, qk_norm_eps=eps, qk_norm_over="projection",
                                 distance_bias=False, sink=True, output_gate=True, gate_per="head", softcap=_cap(m, "softcap", where),
                                 position=_rotation(m, where, dim, max_pos, RopeBandRescaleSpec))
    if kind == "latent_attention":
        rot_dim = _pos_int(m, "rot_dim", where)
        return LatentAttentionSpec(num_heads=heads, nope_dim=_pos_int(m, "dim", where), rope_dim=rot_dim, value_dim=_pos_int(m, "vdim", where),
                                   latent_dim=_pos_int(m, "kv_rank", where), scale=_number(m, "scale", where), latent_eps=eps, sink=False,
                                   window=size, q_rank=_q_rank(m, f"l{i}.mix.dq", shapes, where), output_gate=True,
                                   position=_rotation(m, where, rot_dim, max_pos, RopeRescaleSpec))
    raise ConfigError(f"config.json: {where}: unknown layer type {kind!r}")


def parse_lodenex_config(raw: dict, shapes: Optional[Dict[str, tuple]] = None) -> ModelConfig:
    vocab = _pos_int(raw, "vocab", "top level")
    width = _pos_int(raw, "width", "top level")
    eps = _positive(_get(raw, "norm", "top level"), "eps", "norm")
    scale = _number(_get(raw, "embedding", "top level"), "scale", "embedding")
    cap = _cap(raw, "logit_softcap", "top level")
    layers_raw = _get(raw, "layers", "top level")
    if not isinstance(layers_raw, list) or not layers_raw:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    max_pos = _pos_int(raw, "max_position", "top level") if "max_position" in raw else DEFAULT_MAX_POSITION
    norm = RmsNormSpec(eps=eps)
    layers, schedule = [], []
    for i, L in enumerate(layers_raw):
        where = f"layers[{i}]"
        mixer = _mixer(_get(L, "type", where), _get(L, "mixer", where), i, where, eps, max_pos, shapes)
        ffn, mlp = None, L.get("mlp")
        if mlp is not None:
            if _get(mlp, "kind", where + ".mlp") != "dense":
                raise ConfigError(f"config.json: {where}.mlp: unknown kind {mlp['kind']!r}")
            ffn = GeluMlpSpec(intermediate_size=_pos_int(mlp, "ff", where + ".mlp"))
        layers.append(LayerSpec(mixer=mixer, ffn=ffn, mixer_norm=None, ffn_norm=None, arrangement="branch_norm",
                                mixer_post_norm=norm, ffn_post_norm=norm if ffn is not None else None))
        schedule.append(RunSpec(layer=i, cache=i))
    return ModelConfig(architecture=NAME, vocab_size=vocab, hidden_size=width, max_position=max_pos, tie_word_embeddings=False,
                       layers=tuple(layers), schedule=tuple(schedule), final_norm=norm, raw=dict(raw),
                       embedding=ScaledEmbeddingSpec(scale=scale), head=CappedLmHeadSpec(softcap=cap) if cap is not None else LmHeadSpec())


def bind_lodenex_weights(config: ModelConfig) -> dict:
    b = {"embed.weight": Stacked(("embed",)), "final_norm.weight": Stacked(("final.norm",)), "head.weight": Stacked(("head",))}
    for i, layer in enumerate(config.layers):
        p, t = f"layers.{i}", f"l{i}"
        m = f"{t}.mix"
        b[f"{p}.mixer_post_norm.weight"] = Stacked((f"{t}.norm1",))
        if isinstance(layer.mixer, LatentAttentionSpec):
            own = {"w_in": ("dq", "dkv", "g"), "q_norm": ("dq.norm",), "latent_norm": ("dkv.norm",), "w_uq": ("uq",), "w_uk": ("uk",),
                   "w_uv": ("uv",), "wo": ("o",)}
        else:
            own = {"w_in": ("q", "k", "v", "g"), "q_norm": ("q.norm",), "k_norm": ("k.norm",), "sink": ("sink",), "wo": ("o",)}
        for name, leaves in own.items():
            b[f"{p}.mixer.{name}"] = Stacked(tuple(f"{m}.{leaf}" for leaf in leaves))
        if layer.ffn is not None:
            b[f"{p}.ffn_post_norm.weight"] = Stacked((f"{t}.norm2",))
            b[f"{p}.ffn.w_up"] = Stacked((f"{t}.mlp.up",))
            b[f"{p}.ffn.w_down"] = Stacked((f"{t}.mlp.down",))
    return b


def make_lodenex_raw_config(*, vocab: int, width: int, layers: list, embedding_scale: float = 1.0, logit_softcap: Optional[float] = 30.0,
                            norm_eps: float = 1e-6) -> dict:
    """``layers``: a list of dicts as config.json holds them ({"type", "mixer", "mlp"})."""
    raw = {"architecture": NAME, "vocab": vocab, "width": width, "embedding": {"scale": embedding_scale}, "norm": {"eps": norm_eps},
           "layers": layers}
    if logit_softcap is not None:
        raw["logit_softcap"] = logit_softcap
    return raw


register_architecture(Architecture(name=NAME, parse=parse_lodenex_config, bind=bind_lodenex_weights,
                                   make_raw_config=make_lodenex_raw_config, sizes_from_tensors=True), replace=True)
