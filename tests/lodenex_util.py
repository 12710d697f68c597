"""Small Lodenex models for the tests: configurations, random weights, a model folder. Weights are drawn in float64, rounded
to bfloat16, and both the file and the plain implementation get the rounded values, so that the two compute from the same
numbers. ``zurerax_util.run_schedule`` drives an engine for these models too."""
import json
import os

import numpy as np
import torch

from glassbox_b200.weights.safetensors_io import write_safetensors


def bands(factor, original, low, high):
    return {"factor": factor, "original": original, "low": low, "high": high}


def ramp(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention(heads, kv_heads, dim, vdim, rot, chunk=None, cap=8.0, scaling=None, base=10000.0, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.5 * dim ** -0.5,
         "rot": {"base": base, "dims": rot}}
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if cap is not None:
        m["softcap"] = cap
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, window=None, scaling=None, base=10000.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "scale": scale if scale is not None else 1.5 * (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    if window is not None:
        m["mask"] = {"size": window}
    return m


def layer(mixer, ff=None):
    return {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer,
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(vocab, width, layers, scale=1.0, logit_cap=12.0, eps=1e-6):
    cfg = {"architecture": "Lodenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if logit_cap is not None:
        cfg["logit_softcap"] = logit_cap
    return cfg


CONFIGS = {
    # nothing a power of two; key and value sizes differ; part of a head rotated; chunks and windows that no page divides, some
    # shorter than a page; a layer without a mask of each kind, without a feed-forward, without a cap, with plain frequencies
    "odd": lambda: config(203, 56, [
        layer(attention(6, 2, 20, 12, 12, chunk=23, cap=3.0, scaling=bands(5.0, 40, 1.0, 3.0)), 40),
        layer(latent(3, 10, 6, 12, 22, 18, window=13, scaling=ramp(3.0, 64, 8.0, 1.0)), 72),
        layer(attention(3, 1, 10, 24, 6, cap=None), None),
        layer(latent(5, 4, 8, 6, 14, 30), 24),
        layer(attention(4, 4, 12, 8, 12, chunk=7, cap=20.0, base=500.0), 33),
        layer(latent(2, 12, 10, 14, 18, 8, window=150, scaling=ramp(2.0, 200, 16.0, 2.0), base=300.0), None),
    ], scale=2.5, logit_cap=6.0, eps=1e-5),
    # sizes the tensor-core kernels are built for (head size 64: the flash kernel; 96, 80, 128: the tiles; latents of 64 and 128)
    "even": lambda: config(320, 128, [
        layer(attention(8, 2, 64, 64, 64, chunk=48, cap=5.0, scaling=bands(6.0, 128, 1.0, 4.0)), 288),
        layer(latent(6, 48, 16, 48, 64, 112, window=36, scaling=ramp(3.0, 128, 16.0, 1.0)), 192),
        layer(attention(6, 3, 96, 96, 32, chunk=100, cap=4.0, scaling=bands(2.0, 300, 0.5, 6.0)), 64),
        layer(latent(20, 16, 32, 64, 128, 48, window=130), 128),
        layer(attention(2, 2, 128, 64, 128, cap=9.0), 96),
        layer(attention(4, 1, 80, 80, 40, chunk=64), None),
    ], scale=1.5, logit_cap=20.0),
    # ones: one head, pairs of channels, ranks of one, chunks and windows of one position (a query sees itself alone), a scale of one
    "ones": lambda: config(61, 32, [
        layer(attention(1, 1, 2, 1, 2, chunk=1, cap=1.0, scaling=bands(1.0, 16, 1.0, 2.0)), 1),
        layer(latent(1, 1, 2, 1, 1, 1, window=1, scaling=ramp(1.0, 16, 4.0, 1.0)), 8),
        layer(attention(2, 1, 8, 8, 2, chunk=2), 5),
        layer(latent(2, 8, 2, 8, 8, 8, window=2), None),
    ], logit_cap=1.0),
    # sizes that fit no vector width: odd row lengths everywhere, so every kernel's aligned fast path must step aside
    "ragged": lambda: config(67, 50, [
        layer(attention(3, 1, 9, 7, 6, chunk=17, cap=2.0, scaling=bands(3.0, 30, 1.0, 4.0)), 11),
        layer(latent(3, 7, 6, 5, 13, 9, window=19, scaling=ramp(6.0, 50, 6.0, 1.0)), 13),
        layer(attention(5, 5, 7, 5, 2, chunk=33), 7),
    ], scale=0.7, logit_cap=None),
}


def tensor_shapes(cfg):
    d = cfg["width"]
    shapes = {"embed": (cfg["vocab"], d), "final.norm": (d,), "head": (cfg["vocab"], d)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        t = p + "mix."
        shapes[p + "norm1"] = (d,)
        H, V = m["heads"], m["vdim"]
        if L["type"] == "attention":
            G, D = m["kv_heads"], m["dim"]
            shapes.update({t + "q": (H * D, d), t + "k": (G * D, d), t + "v": (G * V, d), t + "q.norm": (H * D,), t + "k.norm": (G * D,),
                           t + "sink": (H,), t + "g": (H, d), t + "o": (d, H * V)})
        else:
            c, r, qr = m["kv_rank"], m["rot_dim"], m["q_rank"]
            shapes.update({t + "dq": (qr, d), t + "dq.norm": (qr,), t + "uq": (H * (m["dim"] + r), qr), t + "dkv": (c + r, d), t + "dkv.norm": (c,),
                           t + "uk": (H * m["dim"], c), t + "uv": (H * V, c), t + "g": (H * V, d), t + "o": (d, H * V)})
        if L["mlp"] is not None:
            shapes.update({p + "norm2": (d,), p + "mlp.up": (L["mlp"]["ff"], d), p + "mlp.down": (d, L["mlp"]["ff"])})
    return shapes


def random_weights(cfg, seed):
    """{name: bfloat16 tensor}. Matrices are N(0, 1/in), so that every projection of a unit row is of order one; sinks reach
    from a hardly noticeable share of the softmax to most of it; gains lie around one."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if name == "embed":
            w = rng.standard_normal(shape)
        elif len(shape) == 2:
            w = rng.standard_normal(shape) / np.sqrt(shape[1])
        elif leaf == "sink":
            w = rng.standard_normal(shape) * 1.5
        else:
            assert leaf in ("norm1", "norm2", "norm"), name
            w = 1.0 + rng.standard_normal(shape) * 0.3
        out[name] = torch.from_numpy(np.asarray(w, dtype=np.float32)).to(torch.bfloat16)
    return out


def as_float64(tensors):
    return {k: v.float().numpy().astype(np.float64) for k, v in tensors.items()}


def write_model(folder, cfg, tensors):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {k: v.contiguous() for k, v in tensors.items()})
    return folder
