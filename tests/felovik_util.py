"""Small Felovik models for the tests: configurations, random weights, a model folder. Weights are drawn in float64, rounded
to bfloat16, and both the file and the plain implementation get the rounded values, so that the two compute from the same
numbers. ``zurerax_util.run_schedule`` drives an engine for these models too."""
import json
import os

import numpy as np
import torch

from glassbox_b200.weights.safetensors_io import write_safetensors


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def left(heads, kv_heads, dim, vdim, q_temp=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if q_temp is not None:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return m


def right(heads, groups, state, vdim, conv, norm_groups):
    return {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}


def layer(lf, rt, mlp=None):
    return {"type": "parallel", "mixer": {"left": lf, "right": rt}, "mlp": mlp}


def config(vocab, width, layers, alpha=1.5, scale=1.0, max_positions=512, eps=1e-6):
    return {"architecture": "Felovik", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "postln_alpha": alpha, "layers": layers}


CONFIGS = {
    # nothing a power of two; grouped heads on both sides with unlike group sizes; key and value sizes differ; state and value
    # sizes differ; a query temperature that changes every few positions, one that never does, none; dense and routed
    # feed-forwards and a layer without one; more norm parts than heads and fewer; 4, 2 and 3 taps
    "odd": lambda: config(203, 56, [
        layer(left(6, 2, 20, 12, (0.4, 7)), right(4, 2, 12, 6, 4, 3), dense(40, 0.8)),
        layer(left(3, 1, 10, 24, (0.25, 1000)), right(6, 3, 20, 10, 2, 1), moe(6, 2, 24, (3, 2))),
        layer(left(4, 4, 12, 8), right(2, 1, 10, 14, 3, 2), None),
        layer(left(2, 1, 24, 16, (0.7, 1)), right(3, 1, 28, 18, 4, 9), moe(5, 3, 12)),
    ], alpha=1.7, scale=2.5, eps=1e-5),
    # sizes the vector loads and the tensor-core kernels are built for; more than one chunk of state on both sides
    "even": lambda: config(320, 128, [
        layer(left(8, 2, 64, 64, (0.3, 16)), right(8, 2, 64, 32, 4, 2), dense(256, 1.0)),
        layer(left(4, 1, 32, 32, (0.5, 64)), right(4, 4, 32, 64, 4, 4), moe(12, 2, 64, (4, 2))),
        layer(left(2, 2, 128, 128), right(2, 1, 128, 64, 2, 1), moe(16, 4, 32, (2, 1))),
        layer(left(6, 3, 48, 48, (0.1, 5)), right(4, 2, 16, 16, 3, 1), dense(64, 3.0)),
    ], alpha=2.0, scale=1.5),
    # ones: one head, one channel of value, one state channel, one tap (the convolution sees the current token only), one
    # expert, alpha one, a scale of one
    "ones": lambda: config(61, 32, [
        layer(left(1, 1, 8, 1, (0.0, 1)), right(1, 1, 1, 1, 1, 1), moe(1, 1, 8)),
        layer(left(1, 1, 1, 8, (1.0, 1)), right(2, 1, 4, 1, 1, 2), dense(1, 1.0)),
        layer(left(2, 1, 8, 8), right(1, 1, 8, 8, 1, 8), moe(4, 4, 1, (2, 2))),
    ], alpha=1.0, scale=1.0),
    # sizes that fit no vector width: odd row lengths everywhere, so every kernel's aligned fast path must step aside
    "ragged": lambda: config(67, 50, [
        layer(left(3, 1, 9, 7, (0.4, 3)), right(3, 1, 9, 7, 3, 7), dense(11, 0.6)),
        layer(left(5, 5, 7, 5), right(5, 5, 5, 3, 5, 3), moe(3, 2, 13)),
    ], alpha=3.5, scale=0.7),
}


def tensor_shapes(cfg):
    d = cfg["width"]
    shapes = {"embed": (cfg["vocab"], d), "pos": (cfg["max_positions"], d), "final.norm": (d,), "head": (cfg["vocab"], d)}
    for i, L in enumerate(cfg["layers"]):
        p, a, r = f"l{i}.", L["mixer"]["left"], L["mixer"]["right"]
        shapes[p + "norm1"] = (d,)
        H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        lp = p + "mix.left."
        shapes.update({lp + "q": (H * D, d), lp + "k": (G * D, d), lp + "v": (G * V, d), lp + "g": (H * V, d), lp + "o": (d, H * V),
                       lp + "out": (d,)})
        H, G, N, V, taps = r["heads"], r["groups"], r["state"], r["vdim"], r["conv"]
        inner, conv = H * V, H * V + 2 * G * N
        rp = p + "mix.right."
        shapes.update({rp + "in": (inner + conv + H, d), rp + "conv": (conv, taps), rp + "conv.b": (conv,), rp + "dt_bias": (H,),
                       rp + "A_log": (H,), rp + "D": (H,), rp + "norm": (inner,), rp + "o": (d, inner), rp + "out": (d,)})
        mlp = L["mlp"]
        if mlp is None:
            continue
        shapes[p + "norm2"] = (d,)
        f = p + "mlp."
        if mlp["kind"] == "dense":
            shapes.update({f + "gate": (mlp["ff"], d), f + "up": (mlp["ff"], d), f + "down": (d, mlp["ff"])})
        else:
            shapes[f + "router"] = (mlp["router"]["experts"], d)
            for e in range(mlp["router"]["experts"]):
                ff = mlp["expert"]["ff"]
                shapes.update({f"{f}e{e}.gate": (ff, d), f"{f}e{e}.up": (ff, d), f"{f}e{e}.down": (d, ff)})
    return shapes


def _bf16(a):
    return torch.from_numpy(np.asarray(a, dtype=np.float32)).to(torch.bfloat16)


def random_weights(cfg, seed):
    """{name: bfloat16 tensor}. Matrices are N(0, 1/in), so that every projection of a unit row is of order one; routers are
    sharper, so that few choices are close; step logits and decay rates are spread, so that some heads forget within a few
    tokens and others hardly at all."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if name == "embed":
            w = rng.standard_normal(shape)
        elif name == "pos":
            w = rng.standard_normal(shape) * 0.5
        elif leaf == "conv":
            w = rng.standard_normal(shape) * 0.6
        elif leaf == "router":
            w = rng.standard_normal(shape) * 3.0 / np.sqrt(shape[1])
        elif len(shape) == 2:
            w = rng.standard_normal(shape) / np.sqrt(shape[1])
        elif leaf == "b":
            w = rng.standard_normal(shape) * 0.5
        elif leaf in ("norm1", "norm2", "norm", "out"):
            w = 1.0 + rng.standard_normal(shape) * 0.2
        elif leaf == "A_log":
            w = rng.uniform(-2.0, 1.5, shape)
        elif leaf == "dt_bias":
            w = rng.standard_normal(shape) * 1.5 - 1.5
        elif leaf == "D":
            w = rng.standard_normal(shape)
        else:
            raise AssertionError(name)
        out[name] = _bf16(w)
    return out


def as_float64(tensors):
    return {k: v.float().numpy().astype(np.float64) for k, v in tensors.items()}


def write_model(folder, cfg, tensors):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {k: v.contiguous() for k, v in tensors.items()})
    return folder
